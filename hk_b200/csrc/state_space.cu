// State-space mixers (Mamba-2): the recurrence over the rows of every request of a step, its state kept in float32 in the
// request's state slot between steps, and the gated norm behind it.
//
// Per head a matrix state S [N, dv] (zero at a request's start); head h reads B and C of group h / (H / G):
//     dt_t = softplus(dt logit + dt_bias),   S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t
// The columns of S (one per value channel) never mix, and a step's batch is described by a segment table int32
// [n_seg, 3] = (state slot, first row, rows).  x, B and C of a row lie side by side, [x: H dv | B: G N | C: G N], in the
// storage type (what the short convolution before wrote); decays, step sizes, state and sums are float32.
//
// The state of a slot is stored [H, dv, N]: a column's N entries are neighbours, so the lanes that share a column read and
// write whole lines.
#include "common.cuh"

namespace {

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }

template <int BYTES>
__device__ __forceinline__ void cp_async(void* dst, const void* src) {
  if (BYTES == 16)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
  else
    asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "n"(BYTES) : "memory");
}

// four neighbours of shared memory as floats
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                     __uint_as_float(v.y & 0xffff0000u));
}

}  // namespace

// The sums over the L lanes that share CPT columns, as a butterfly: while a lane carries several columns, half of them go to
// the partner.  Afterwards a lane holds, in acc[0], the sum of the column whose number is returned.
template <int L, int CPT>
__device__ __forceinline__ int sum_over_lanes(float* acc, int sub) {
  int mine = 0, at = L >> 1;
#pragma unroll
  for (int width = CPT >> 1; width > 0; width >>= 1) {
    const bool upper = (sub & at) != 0;
#pragma unroll
    for (int k = 0; k < width; ++k) {
      const float keep = upper ? acc[k + width] : acc[k], give = upper ? acc[k] : acc[k + width];
      acc[k] = keep + __shfl_xor_sync(0xffffffffu, give, at);
    }
    if (upper) mine += width;
    at >>= 1;
  }
#pragma unroll
  for (int o = L / 2 / CPT; o > 0; o >>= 1) acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], o);
  return mine;
}
// one lane of those that hold the same column
template <int L, int CPT>
__device__ __forceinline__ bool writes_sum(int sub) { return (sub & (L / CPT - 1)) == 0; }

// ------------------------------------------------------------------ the walk, token by token
// A block of 128 threads owns `cols` = 128 / L * CPT columns of one head's state for one segment.  A column's entries are
// spread over L lanes, RPT per lane, in registers: lane `sub` holds the entries 4 (q L + sub) .. + 3 for q < RPT / 4, and a
// lane group holds CPT columns (they share every load of B and C).  Rows arrive in chunks of `chunk` tokens through a
// two-stage cp.async ring in the storage type; the head's two scalars of a token (decay, step size) are made once per
// chunk.  The chain that the next token waits for is one multiply and one fused multiply-add per state entry; the
// read-out's sums over the L lanes hang off it, as a butterfly that halves the columns a lane carries while it can.
template <typename T, int L, int RPT, int CPT>
__global__ void __launch_bounds__(128)
state_space_walk_kernel(const T* __restrict__ xbc, long long ldx, const float* __restrict__ dt, long long ldt,
                        const float* __restrict__ dt_bias, const float* __restrict__ a_log, const float* __restrict__ skip,
                        const int* __restrict__ segs, float* __restrict__ state, float* __restrict__ y, int H, int G, int N, int dv,
                        int chunk, int vec) {
  constexpr int P = L * RPT;
  constexpr int COLS = 128 / L * CPT;
  constexpr int R = 2 * P + COLS;                  // elements of a token in a stage: B, C, the block's values
  extern __shared__ __align__(16) uint8_t smem_raw[];
  T* rows = reinterpret_cast<T*>(smem_raw);                                     // [2][chunk][R]
  float* raw_dt = reinterpret_cast<float*>(rows + (size_t)2 * chunk * R);       // [2][chunk] the head's step-size logits
  float2* scal = reinterpret_cast<float2*>(raw_dt + 2 * chunk);                 // [chunk] (decay, step size)
  const int seg = blockIdx.x / H, h = blockIdx.x % H;
  const int slot = segs[seg * 3], row0 = segs[seg * 3 + 1], count = segs[seg * 3 + 2];
  const int col0 = blockIdx.y * COLS, ncols = min(COLS, dv - col0);
  const int tid = threadIdx.x, sub = tid % L, c0 = (tid / L) * CPT;
  const float bias = dt_bias[h], rate = expf(a_log[h]), dskip = skip[h];

  float S[CPT][RPT];
  float* sp = state + (((size_t)slot * H + h) * dv + col0 + c0) * N;
  const bool whole = (N & 3) == 0;
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int q = 0; q < RPT / 4; ++q) {
      const int i = 4 * (q * L + sub);
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c0 + c < ncols) {
        const float* p = sp + (size_t)c * N + i;
        if (whole) {
          if (i < N) v = *reinterpret_cast<const float4*>(p);
        } else {
          if (i < N) v.x = p[0];
          if (i + 1 < N) v.y = p[1];
          if (i + 2 < N) v.z = p[2];
          if (i + 3 < N) v.w = p[3];
        }
      }
      S[c][4 * q] = v.x; S[c][4 * q + 1] = v.y; S[c][4 * q + 2] = v.z; S[c][4 * q + 3] = v.w;
    }
  if (N < P || ncols < COLS) {                     // what no copy below ever touches: the padding must not hold NaN patterns
    for (int i = tid; i < 2 * chunk * R; i += 128) rows[i] = from_f32<T>(0.f);
    __syncthreads();
  }

  const T* xs = xbc + (size_t)row0 * ldx + (size_t)h * dv + col0;
  const T* bs = xbc + (size_t)row0 * ldx + (size_t)H * dv + (size_t)(h / (H / G)) * N;
  const T* cs = bs + (size_t)G * N;
  const float* ds = dt + (size_t)row0 * ldt + h;
  auto fetch = [&](int c) {                        // chunk c -> stage c & 1
    const int t0 = c * chunk, tc = min(chunk, count - t0);
    T* dst = rows + (size_t)(c & 1) * chunk * R;
    if (vec) {
      constexpr int V = 16 / sizeof(T);
      const int nb = N / V, nx = ncols / V, per = 2 * nb + nx;
      for (int i = tid; i < tc * per; i += 128) {
        const int t = i / per, p = i - t * per;
        const size_t src = (size_t)(t0 + t) * ldx;
        T* d = dst + (size_t)t * R;
        if (p < nb) cp_async<16>(d + p * V, bs + src + p * V);
        else if (p < 2 * nb) cp_async<16>(d + P + (p - nb) * V, cs + src + (p - nb) * V);
        else cp_async<16>(d + 2 * P + (p - 2 * nb) * V, xs + src + (p - 2 * nb) * V);
      }
    } else {
      const int per = 2 * N + ncols;
      for (int i = tid; i < tc * per; i += 128) {
        const int t = i / per, p = i - t * per;
        const size_t src = (size_t)(t0 + t) * ldx;
        T* d = dst + (size_t)t * R;
        if (p < N) d[p] = bs[src + p];
        else if (p < 2 * N) d[P + p - N] = cs[src + p - N];
        else d[2 * P + p - 2 * N] = xs[src + p - 2 * N];
      }
    }
    for (int t = tid; t < tc; t += 128) cp_async<4>(raw_dt + (c & 1) * chunk + t, ds + (size_t)(t0 + t) * ldt);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int nchunks = (count + chunk - 1) / chunk;
  float* yp = y + (size_t)row0 * H * dv + (size_t)h * dv + col0 + c0;
  const size_t ystep = (size_t)H * dv;
  fetch(0);
  for (int c = 0; c < nchunks; ++c) {
    if (c + 1 < nchunks) {
      fetch(c + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const int tc = min(chunk, count - c * chunk);
    for (int t = tid; t < tc; t += 128) {
      const float step = softplus_f(raw_dt[(c & 1) * chunk + t] + bias);
      scal[t] = make_float2(expf(-rate * step), step);
    }
    __syncthreads();
    const T* buf = rows + (size_t)(c & 1) * chunk * R;
#pragma unroll 2
    for (int t = 0; t < tc; ++t) {
      const T* tok = buf + (size_t)t * R;
      const float2 ds_t = scal[t];
      float x[CPT], u[CPT], acc[CPT];
#pragma unroll
      for (int cc = 0; cc < CPT; ++cc) {
        x[cc] = to_f32<T>(tok[2 * P + c0 + cc]);
        u[cc] = ds_t.y * x[cc];
        acc[cc] = 0.f;
      }
#pragma unroll
      for (int q = 0; q < RPT / 4; ++q) {
        const float4 b = load4(tok + 4 * (q * L + sub));
        const float4 g = load4(tok + P + 4 * (q * L + sub));
#pragma unroll
        for (int cc = 0; cc < CPT; ++cc) {
          float* s = S[cc] + 4 * q;
          s[0] = fmaf(b.x, u[cc], ds_t.x * s[0]);
          s[1] = fmaf(b.y, u[cc], ds_t.x * s[1]);
          s[2] = fmaf(b.z, u[cc], ds_t.x * s[2]);
          s[3] = fmaf(b.w, u[cc], ds_t.x * s[3]);
          acc[cc] = fmaf(g.x, s[0], acc[cc]);
          acc[cc] = fmaf(g.y, s[1], acc[cc]);
          acc[cc] = fmaf(g.z, s[2], acc[cc]);
          acc[cc] = fmaf(g.w, s[3], acc[cc]);
        }
      }
      const int mine = sum_over_lanes<L, CPT>(acc, sub);
      float xm = x[0];
#pragma unroll
      for (int k = 1; k < CPT; ++k) xm = mine == k ? x[k] : xm;
      if (writes_sum<L, CPT>(sub) && c0 + mine < ncols) yp[(size_t)t * ystep + mine] = fmaf(dskip, xm, acc[0]);
    }
    yp += (size_t)tc * ystep;
    __syncthreads();                               // the stage and the scalars may be filled again
  }
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int q = 0; q < RPT / 4; ++q) {
      const int i = 4 * (q * L + sub);
      if (c0 + c < ncols) {
        float* p = sp + (size_t)c * N + i;
        if (whole) {
          if (i < N) *reinterpret_cast<float4*>(p) = make_float4(S[c][4 * q], S[c][4 * q + 1], S[c][4 * q + 2], S[c][4 * q + 3]);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (i + e < N) p[e] = S[c][4 * q + e];
        }
      }
    }
}

// A step of single tokens (a decode step): the same arithmetic on one row per segment, without the ring and its barriers:
// everything a thread needs is asked for at once, straight into registers.  Every segment has one row.
template <typename T, int L, int RPT, int CPT>
__global__ void __launch_bounds__(128)
state_space_step_kernel(const T* __restrict__ xbc, long long ldx, const float* __restrict__ dt, long long ldt,
                        const float* __restrict__ dt_bias, const float* __restrict__ a_log, const float* __restrict__ skip,
                        const int* __restrict__ segs, float* __restrict__ state, float* __restrict__ y, int H, int G, int N, int dv) {
  constexpr int COLS = 128 / L * CPT;
  const int seg = blockIdx.x / H, h = blockIdx.x % H;
  const int slot = segs[seg * 3], row = segs[seg * 3 + 1];
  const int tid = threadIdx.x, sub = tid % L, c0 = blockIdx.y * COLS + (tid / L) * CPT;
  float* sp = state + (((size_t)slot * H + h) * dv + c0) * N;
  const T* xs = xbc + (size_t)row * ldx + (size_t)h * dv + c0;
  const T* bs = xbc + (size_t)row * ldx + (size_t)H * dv + (size_t)(h / (H / G)) * N;
  const T* cs = bs + (size_t)G * N;
  float4 S[CPT][RPT / 4], b[RPT / 4], g[RPT / 4];
  float x[CPT], u[CPT], acc[CPT];
  bool in[RPT / 4];                                // N is a multiple of 4: four entries at a time exist or do not
#pragma unroll
  for (int q = 0; q < RPT / 4; ++q) {
    const int i = 4 * (q * L + sub);
    in[q] = i < N;
#pragma unroll
    for (int c = 0; c < CPT; ++c)
      S[c][q] = in[q] && c0 + c < dv ? *reinterpret_cast<const float4*>(sp + (size_t)c * N + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    b[q] = in[q] ? make_float4(to_f32<T>(bs[i]), to_f32<T>(bs[i + 1]), to_f32<T>(bs[i + 2]), to_f32<T>(bs[i + 3])) : make_float4(0.f, 0.f, 0.f, 0.f);
    g[q] = in[q] ? make_float4(to_f32<T>(cs[i]), to_f32<T>(cs[i + 1]), to_f32<T>(cs[i + 2]), to_f32<T>(cs[i + 3])) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const float step = softplus_f(dt[(size_t)row * ldt + h] + dt_bias[h]);
  const float decay = expf(-expf(a_log[h]) * step), dskip = skip[h];
#pragma unroll
  for (int c = 0; c < CPT; ++c) {
    x[c] = c0 + c < dv ? to_f32<T>(xs[c]) : 0.f;
    u[c] = step * x[c];
    acc[c] = 0.f;
  }
#pragma unroll
  for (int q = 0; q < RPT / 4; ++q)
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
      float4& s = S[c][q];
      s.x = fmaf(b[q].x, u[c], decay * s.x);
      s.y = fmaf(b[q].y, u[c], decay * s.y);
      s.z = fmaf(b[q].z, u[c], decay * s.z);
      s.w = fmaf(b[q].w, u[c], decay * s.w);
      acc[c] = fmaf(g[q].x, s.x, acc[c]);
      acc[c] = fmaf(g[q].y, s.y, acc[c]);
      acc[c] = fmaf(g[q].z, s.z, acc[c]);
      acc[c] = fmaf(g[q].w, s.w, acc[c]);
      if (in[q] && c0 + c < dv) *reinterpret_cast<float4*>(sp + (size_t)c * N + 4 * (q * L + sub)) = s;
    }
  const int mine = sum_over_lanes<L, CPT>(acc, sub);
  float xm = x[0];
#pragma unroll
  for (int k = 1; k < CPT; ++k) xm = mine == k ? x[k] : xm;
  if (writes_sum<L, CPT>(sub) && c0 + mine < dv) y[(size_t)row * H * dv + (size_t)h * dv + c0 + mine] = fmaf(dskip, xm, acc[0]);
}

template <typename T, int L, int RPT, int CPT>
static int walk_launch(const T* xbc, long long ldx, const float* dt, long long ldt, const float* dt_bias, const float* a_log,
                       const float* skip, const int* segs, int n_seg, float* state, float* y, int H, int G, int N, int dv,
                       int single, cudaStream_t s) {
  constexpr int COLS = 128 / L * CPT, R = 2 * L * RPT + COLS;
  dim3 grid((unsigned)(n_seg * H), (unsigned)((dv + COLS - 1) / COLS));
  if (single && (N & 3) == 0)
    return hk_launch(state_space_step_kernel<T, L, RPT, CPT>, grid, dim3(128), 0, s, xbc, ldx, dt, ldt, dt_bias, a_log, skip, segs, state, y,
                     H, G, N, dv);
  constexpr int V = 16 / sizeof(T);
  const int inner = H * dv;
  const int vec = ((uintptr_t)xbc & 15) == 0 && ldx % V == 0 && inner % V == 0 && N % V == 0 && dv % V == 0 && COLS % V == 0;
  int chunk = 16;
  auto bytes = [&](int c) { return (size_t)2 * c * R * sizeof(T) + 2 * c * sizeof(float) + c * sizeof(float2); };
  while (chunk > 2 && bytes(chunk) > 48 * 1024) chunk >>= 1;
  const size_t smem = bytes(chunk);
  static HkSmemCache cache;
  if (int e = hk_allow_smem(state_space_walk_kernel<T, L, RPT, CPT>, smem, cache)) return e;
  return hk_launch(state_space_walk_kernel<T, L, RPT, CPT>, grid, dim3(128), smem, s, xbc, ldx, dt, ldt, dt_bias, a_log, skip, segs,
                   state, y, H, G, N, dv, chunk, vec);
}

// Four columns a lane group where the blocks fill the SMs twice, two where they do not (a column's entries spread over L
// lanes either way): the layout of the sums does not depend on it.
template <typename T>
static int walk(const T* xbc, long long ldx, const float* dt, long long ldt, const float* dt_bias, const float* a_log,
                const float* skip, const int* segs, int n_seg, float* state, float* y, int H, int G, int N, int dv, int single,
                cudaStream_t s) {
#define WALK(L, RPT, CPT) walk_launch<T, L, RPT, CPT>(xbc, ldx, dt, ldt, dt_bias, a_log, skip, segs, n_seg, state, y, H, G, N, dv, single, s)
#define WALK_ANY(L, RPT)                                                                                 \
  do {                                                                                                   \
    const bool many = (long long)n_seg * H * ((dv + 128 / L * 4 - 1) / (128 / L * 4)) >= 2 * 148;        \
    return many ? WALK(L, RPT, 4) : WALK(L, RPT, 2);                                                     \
  } while (0)
  if (N <= 32) WALK_ANY(8, 4);
  if (N <= 64) WALK_ANY(8, 8);
  if (N <= 128) WALK_ANY(16, 8);
  if (N <= 256) WALK_ANY(32, 8);
  if (N <= 512) return WALK(32, 16, 2);
  if (N <= 1024) return WALK(32, 32, 2);
  return HK_ERR_UNSUPPORTED;
#undef WALK_ANY
#undef WALK
}

// xbc [n, >= H dv + 2 G N] float32 or bf16 (row stride ldx); dt float32 [n, H] (row stride ldt); dt_bias, a_log, skip float32
// [H]; state float32 [slots, H, dv, N]; y float32 [n, H dv].  single = 1 says that every segment has one row.
HK_API int hk_state_space_walk(const void* xbc, int dtype, long long ldx, const float* dt, long long ldt, const float* dt_bias,
                               const float* a_log, const float* skip, const int* segs, int n_seg, int n_rows, float* state, float* y,
                               int H, int G, int N, int dv, int single, void* stream) {
  if (n_seg <= 0 || n_rows <= 0) return 0;
  if (H < 1 || G < 1 || H % G || N < 1 || N > 1024 || dv < 1 || ((uintptr_t)state & 15)) return HK_ERR_UNSUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == HK_F32)
    return walk<float>((const float*)xbc, ldx, dt, ldt, dt_bias, a_log, skip, segs, n_seg, state, y, H, G, N, dv, single, s);
  if (dtype == HK_BF16)
    return walk<bf16>((const bf16*)xbc, ldx, dt, ldt, dt_bias, a_log, skip, segs, n_seg, state, y, H, G, N, dv, single, s);
  return HK_ERR_UNSUPPORTED;
}

// ------------------------------------------------------------------ the walk, a chunk of tokens at a time (bf16 inputs)
// The same recurrence for prompt portions as matrix products over chunks of 64 tokens, on mma.sync.  With the chunk's
// cumulative log decays c_t (c_0 the first token's own) and its start state S_0, in exact arithmetic
//     y_t = e^(c_t) S_0^T C_t + sum_(s <= t) e^(c_t - c_s) dt_s (C_t . B_s) x_s + D x_t
//     S   = e^(c_last) S_0 + sum_s B_s (e^(c_last - c_s) dt_s x_s)^T
// x, B and C are bf16 as they come and enter the products as they are; every float32 factor (the state, the weighted x, the
// decayed scores) is cut into three bf16 numbers whose sum is the float32 number to its last bit or two, one product each,
// with float32 sums.  The state stays in float32 registers from a portion's first chunk to its last.
//
// A block owns DVB value columns of one head for one segment and walks its chunks in order, the next chunk's rows on their
// way through cp.async meanwhile.  Two groups of eight warps work side by side: while the outputs of chunk c are made from
// the start state S_c, the other group makes S_(c+1) and lays its pieces out for everyone (two buffers), so a chunk costs
// the longer of the two, and one barrier of the block.
//   * outputs: warps r and r + 4 share the tokens 16 r .. 16 r + 15: each takes half of the entries of C S_c and every other
//     16-token block of the scores; the second hands its sums to the first through shared memory;
//   * state: a warp holds its share of the state's tiles (16 entries x 8 columns) in registers from a portion's first chunk
//     to its last; the group first lays out the weighted x in pieces.
namespace {

constexpr int CQ = 64;      // tokens of a chunk

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16_or_zero(void* dst, const void* src, bool valid) {
  const int bytes = valid ? 16 : 0;   // 0 source bytes: the 16 destination bytes are zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldmatrix_x2_trans(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 2^x for x <= 0 (what falls below the smallest normal number is 0)
__device__ __forceinline__ float exp2_f(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
// two float32 numbers as three pairs of bf16 whose sums they are
__device__ __forceinline__ void split3(float a, float b, uint32_t* out) {
#pragma unroll
  for (int p = 0; p < 3; ++p) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    out[p] = *reinterpret_cast<const uint32_t*>(&v);
    a -= __uint_as_float(out[p] << 16);
    b -= __uint_as_float(out[p] & 0xffff0000u);
  }
}

template <int NT, int DVB>
struct ChunkShape {
  static constexpr int LDN = NT + 8, LDX = DVB + 8;              // padded rows: an odd number of 16-byte pieces
  static constexpr int RT = NT / 16;                             // state tiles of 16 entries
  static constexpr int MT = RT > 8 ? RT / 8 : 1;                 // of which a warp holds MT ...
  static constexpr int CP = RT < 8 ? 8 / RT : 1;                 // ... in 1 / CP of the columns,
  static constexpr int NC = DVB / 8 / CP;                        // NC tiles of 8
  static constexpr int NY = DVB / 8;                             // column tiles of the outputs
  // the sums that change hands go where the pair's 16 rows of C lay, if they fit there
  static constexpr bool OVER_C = 16 * LDN * 2 >= 16 * DVB * 4;
  static constexpr size_t BC = (size_t)2 * 2 * CQ * LDN, X = (size_t)2 * CQ * LDX, XW = (size_t)3 * CQ * LDX, SS = (size_t)3 * NT * LDX;
  static constexpr size_t SMEM = (BC + X + XW + 2 * SS) * sizeof(bf16) + 2 * CQ * sizeof(float2) + (OVER_C ? 0 : (size_t)CQ * DVB * sizeof(float));
  static_assert(NC >= 1 && SMEM <= 227 * 1024, "the block's shared memory");
};

// barriers: 0 the block, 1..4 the pairs of output warps, 5 the state group
__device__ __forceinline__ void group_sync(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }

}  // namespace

template <int NT, int DVB>
__global__ void __launch_bounds__(512, 1)
state_space_chunks_kernel(const bf16* __restrict__ xbc, long long ldx, const float* __restrict__ dt, long long ldt,
                          const float* __restrict__ dt_bias, const float* __restrict__ a_log, const float* __restrict__ skip,
                          const int* __restrict__ segs, float* __restrict__ state, float* __restrict__ y, int H, int G, int N, int dv) {
  using K = ChunkShape<NT, DVB>;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* bs = reinterpret_cast<bf16*>(smem_raw);       // [2][CQ][LDN]
  bf16* cs = bs + 2 * CQ * K::LDN;                    // [2][CQ][LDN]
  bf16* xs = cs + 2 * CQ * K::LDN;                    // [2][CQ][LDX]
  bf16* xw = xs + K::X;                               // [3][CQ][LDX] the weighted x in three pieces
  bf16* ss = xw + K::XW;                              // [2][3][NT][LDX] a chunk's start state in three pieces
  float2* scal = reinterpret_cast<float2*>(ss + 2 * K::SS);     // [2][CQ] (cumulative log2 decay, step size)
  float* hand = reinterpret_cast<float*>(scal + 2 * CQ);        // [4][16][DVB], unless those lie over C

  const int seg = blockIdx.x / H, h = blockIdx.x % H;
  const int slot = segs[seg * 3], row0 = segs[seg * 3 + 1], count = segs[seg * 3 + 2];
  const int col0 = blockIdx.y * DVB, ncols = min(DVB, dv - col0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qr = lane >> 2, qt = lane & 3, mi = lane >> 3, r8 = lane & 7;
  const int nchunks = (count + CQ - 1) / CQ;

  const bf16* xg = xbc + (size_t)row0 * ldx + (size_t)h * dv + col0;
  const bf16* bg = xbc + (size_t)row0 * ldx + (size_t)H * dv + (size_t)(h / (H / G)) * N;
  const bf16* cg = bg + (size_t)G * N;
  auto fetch = [&](int c) {                           // chunk c -> stage c & 1, rows and columns that do not exist as zeros
    const int t0 = c * CQ, tc = min(CQ, count - t0);
    bf16* db = bs + (size_t)(c & 1) * CQ * K::LDN;
    bf16* dc = cs + (size_t)(c & 1) * CQ * K::LDN;
    bf16* dx = xs + (size_t)(c & 1) * CQ * K::LDX;
    for (int e = tid; e < CQ * (NT / 8); e += 512) {
      const int t = e / (NT / 8), p = (e % (NT / 8)) * 8;
      const bool ok = t < tc && p < N;
      const size_t src = ok ? (size_t)(t0 + t) * ldx + p : 0;
      cp_async16_or_zero(db + t * K::LDN + p, bg + src, ok);
      cp_async16_or_zero(dc + t * K::LDN + p, cg + src, ok);
    }
    for (int e = tid; e < CQ * (DVB / 8); e += 512) {
      const int t = e / (DVB / 8), p = (e % (DVB / 8)) * 8;
      const bool ok = t < tc && p < ncols;
      cp_async16_or_zero(dx + t * K::LDX + p, xg + (ok ? (size_t)(t0 + t) * ldx + p : 0), ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto next_chunk = [&](int c) {                      // everything of chunk c is there, and chunk c + 1 is asked for
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (c + 1 < nchunks) fetch(c + 1);
  };
  fetch(0);

  if (warp < 8) {
    // ---------------------------------------------------------------- outputs
    const int rg = warp & 3, side = warp >> 2;        // tokens 16 rg .., which half of the work
    const float dskip = skip[h];
    const size_t ystep = (size_t)H * dv;
    float* yp = y + (size_t)row0 * ystep + (size_t)h * dv + col0;
    for (int c = 0; c < nchunks; ++c) {
      next_chunk(c);
      const bf16* bt = bs + (size_t)(c & 1) * CQ * K::LDN;
      bf16* ct = cs + (size_t)(c & 1) * CQ * K::LDN;
      const bf16* xt = xs + (size_t)(c & 1) * CQ * K::LDX;
      const float2* sc = scal + (c & 1) * CQ;
      // C S_c over this side's entries; the scores C B^T of the blocks side and side + 2 (of those up to the tokens')
      float acc[K::NY][4], g[2][2][4];
#pragma unroll
      for (int n = 0; n < K::NY; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) g[j][i][e] = 0.f;
      const bf16* ca = ct + (rg * 16 + r8 + (mi & 1) * 8) * K::LDN + (mi >> 1) * 8;
      const bf16* bb = bt + (side * 16 + (mi >> 1) * 8 + r8) * K::LDN + (mi & 1) * 8;
      const bf16* sb = ss + (size_t)(c & 1) * K::SS + (size_t)((mi & 1) * 8 + r8) * K::LDX + (mi >> 1) * 8;
#pragma unroll
      for (int k = 0; k < NT / 16; ++k) {
        uint32_t a[4];
        ldmatrix_x4(a, ca + k * 16);
        if ((k >= NT / 32) == (side == 1)) {
#pragma unroll
          for (int p = 0; p < 3; ++p)
#pragma unroll
            for (int np = 0; np < K::NY / 2; ++np) {
              uint32_t b[4];
              ldmatrix_x4_trans(b, sb + ((size_t)p * NT + k * 16) * K::LDX + np * 16);
              mma_bf16(acc[2 * np], a, b[0], b[1]);
              mma_bf16(acc[2 * np + 1], a, b[2], b[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
          if (2 * j + side <= rg) {
            uint32_t b[4];
            ldmatrix_x4(b, bb + j * 32 * K::LDN + k * 16);
            mma_bf16(g[j][0], a, b[0], b[1]);
            mma_bf16(g[j][1], a, b[2], b[3]);
          }
      }
      if (K::OVER_C) group_sync(1 + rg, 64);          // both warps have read the pair's rows of C
      const int t0 = rg * 16 + qr;
      const float cum0 = sc[t0].x, cum1 = sc[t0 + 8].x;
      const float f0 = exp2_f(cum0), f1 = exp2_f(cum1);
#pragma unroll
      for (int n = 0; n < K::NY; ++n) {
        acc[n][0] *= f0;
        acc[n][1] *= f0;
        acc[n][2] *= f1;
        acc[n][3] *= f1;
      }
      const bf16* xb = xt + (side * 16 + (mi & 1) * 8 + r8) * K::LDX + (mi >> 1) * 8;
#pragma unroll
      for (int j = 0; j < 2; ++j)
        if (2 * j + side <= rg) {
          uint32_t piece[4][3];                       // the decayed scores of 16 x 16 as an A fragment, in three pieces
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int s = (2 * j + side) * 16 + i * 8 + 2 * qt;
            const float4 sw = *reinterpret_cast<const float4*>(sc + s);     // two tokens: (decay, step), (decay, step)
            const float m0 = s <= t0 ? g[j][i][0] * (exp2_f(cum0 - sw.x) * sw.y) : 0.f;
            const float m1 = s + 1 <= t0 ? g[j][i][1] * (exp2_f(cum0 - sw.z) * sw.w) : 0.f;
            const float m2 = s <= t0 + 8 ? g[j][i][2] * (exp2_f(cum1 - sw.x) * sw.y) : 0.f;
            const float m3 = s + 1 <= t0 + 8 ? g[j][i][3] * (exp2_f(cum1 - sw.z) * sw.w) : 0.f;
            split3(m0, m1, piece[2 * i]);
            split3(m2, m3, piece[2 * i + 1]);
          }
          uint32_t b[K::NY / 2][4];
#pragma unroll
          for (int np = 0; np < K::NY / 2; ++np) ldmatrix_x4_trans(b[np], xb + j * 32 * K::LDX + np * 16);
#pragma unroll
          for (int p = 0; p < 3; ++p) {
            const uint32_t a[4] = {piece[0][p], piece[1][p], piece[2][p], piece[3][p]};
#pragma unroll
            for (int np = 0; np < K::NY / 2; ++np) {
              mma_bf16(acc[2 * np], a, b[np][0], b[np][1]);
              mma_bf16(acc[2 * np + 1], a, b[np][2], b[np][3]);
            }
          }
        }
      // the second warp's sums to the first, a lane's own numbers side by side over the lanes
      float* hp = K::OVER_C ? reinterpret_cast<float*>(ct + rg * 16 * K::LDN) : hand + rg * 16 * DVB;
      if (side == 1) {
#pragma unroll
        for (int n = 0; n < K::NY; ++n)
          *reinterpret_cast<float4*>(hp + (n * 32 + lane) * 4) = make_float4(acc[n][0], acc[n][1], acc[n][2], acc[n][3]);
      }
      group_sync(1 + rg, 64);
      if (side == 0) {
        const int left = count - c * CQ;              // tokens from the chunk's first on
#pragma unroll
        for (int n = 0; n < K::NY; ++n) {
          const float4 o = *reinterpret_cast<const float4*>(hp + (n * 32 + lane) * 4);
          const float v[4] = {acc[n][0] + o.x, acc[n][1] + o.y, acc[n][2] + o.z, acc[n][3] + o.w};
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int t = t0 + 8 * i, d = n * 8 + 2 * qt;
            if (t < left && d < ncols) {
              const uint32_t x = *reinterpret_cast<const uint32_t*>(xt + t * K::LDX + d);
              *reinterpret_cast<float2*>(yp + (size_t)(c * CQ + t) * ystep + d) =
                  make_float2(fmaf(dskip, __uint_as_float(x << 16), v[2 * i]), fmaf(dskip, __uint_as_float(x & 0xffff0000u), v[2 * i + 1]));
            }
          }
        }
      }
    }
    return;
  }

  // ------------------------------------------------------------------ the state
  const int sw = warp - 8, st = tid - 256;
  // this warp's state tiles: rows (entries) st_row + 128 m + .., columns st_col + 8 c + ..
  const int st_row = (sw % (K::RT < 8 ? K::RT : 8)) * 16, st_col = (K::RT < 8 ? sw / K::RT : 0) * K::NC * 8;
  float* sp = state + (((size_t)slot * H + h) * dv + col0) * N;
  float S[K::MT][K::NC][4];
#pragma unroll
  for (int m = 0; m < K::MT; ++m)
#pragma unroll
    for (int c = 0; c < K::NC; ++c)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = st_row + 128 * m + qr + 8 * (e >> 1), d = st_col + 8 * c + 2 * qt + (e & 1);
        S[m][c][e] = n < N && d < ncols ? sp[(size_t)d * N + n] : 0.f;
      }
  auto publish = [&](int c) {                         // S_c in three pieces, for the read-out of chunk c
#pragma unroll
    for (int m = 0; m < K::MT; ++m)
#pragma unroll
      for (int n = 0; n < K::NC; ++n)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          uint32_t piece[3];
          split3(S[m][n][2 * i], S[m][n][2 * i + 1], piece);
          bf16* d = ss + (size_t)(c & 1) * K::SS + (size_t)(st_row + 128 * m + qr + 8 * i) * K::LDX + st_col + 8 * n + 2 * qt;
#pragma unroll
          for (int p = 0; p < 3; ++p) *reinterpret_cast<uint32_t*>(d + (size_t)p * NT * K::LDX) = piece[p];
        }
  };
  // the group's first warp makes a chunk's scalars: lane l the tokens 2 l and 2 l + 1, their logits asked for a chunk ahead
  const float bias = dt_bias[h], rate2 = expf(a_log[h]) * 1.4426950408889634f;
  float raw[2] = {0.f, 0.f};
  auto ask = [&](int c) {
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int t = c * CQ + 2 * lane + u;
      raw[u] = t < count ? dt[(size_t)(row0 + t) * ldt + h] : 0.f;
    }
  };
  auto scalars = [&](int c) {
    float step[2], la[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      step[u] = c * CQ + 2 * lane + u < count ? softplus_f(raw[u] + bias) : 0.f;
      la[u] = -rate2 * step[u];
    }
    float run = la[0] + la[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += v;
    }
    float before = __shfl_up_sync(0xffffffffu, run, 1);
    if (lane == 0) before = 0.f;
    scal[(c & 1) * CQ + 2 * lane] = make_float2(before + la[0], step[0]);
    scal[(c & 1) * CQ + 2 * lane + 1] = make_float2(run, step[1]);
  };
  if (sw == 0) {
    ask(0);
    scalars(0);
  }
  publish(0);
  for (int c = 0; c < nchunks; ++c) {
    next_chunk(c);
    if (sw == 0 && c + 1 < nchunks) ask(c + 1);
    const bf16* bt = bs + (size_t)(c & 1) * CQ * K::LDN;
    const bf16* xt = xs + (size_t)(c & 1) * CQ * K::LDX;
    const float2* sc = scal + (c & 1) * CQ;
    const float last = sc[CQ - 1].x;
#pragma unroll
    for (int i = 0; i < CQ * (DVB / 2) / 256; ++i) {
      const int e = st + 256 * i, t = e / (DVB / 2), d = (e % (DVB / 2)) * 2;
      const uint32_t v = *reinterpret_cast<const uint32_t*>(xt + t * K::LDX + d);
      const float w = exp2_f(last - sc[t].x) * sc[t].y;
      uint32_t piece[3];
      split3(w * __uint_as_float(v << 16), w * __uint_as_float(v & 0xffff0000u), piece);
#pragma unroll
      for (int p = 0; p < 3; ++p) *reinterpret_cast<uint32_t*>(xw + (size_t)p * CQ * K::LDX + t * K::LDX + d) = piece[p];
    }
    group_sync(5, 256);                               // the weighted x is there
    const float keep = exp2_f(last);
#pragma unroll
    for (int m = 0; m < K::MT; ++m)
#pragma unroll
      for (int n = 0; n < K::NC; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[m][n][e] *= keep;
    const bf16* ba = bt + ((mi >> 1) * 8 + r8) * K::LDN + st_row + (mi & 1) * 8;
    const bf16* wb = xw + ((mi & 1) * 8 + r8) * K::LDX + st_col + (mi >> 1) * 8;
#pragma unroll
    for (int k = 0; k < CQ / 16; ++k) {
      uint32_t a[K::MT][4];
#pragma unroll
      for (int m = 0; m < K::MT; ++m) ldmatrix_x4_trans(a[m], ba + k * 16 * K::LDN + 128 * m);
#pragma unroll
      for (int p = 0; p < 3; ++p) {
        if (K::NC == 1) {
          uint32_t b[2];
          ldmatrix_x2_trans(b, xw + ((size_t)p * CQ + k * 16 + (lane & 15)) * K::LDX + st_col);
#pragma unroll
          for (int m = 0; m < K::MT; ++m) mma_bf16(S[m][0], a[m], b[0], b[1]);
        } else {
#pragma unroll
          for (int np = 0; np < K::NC / 2; ++np) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, wb + ((size_t)p * CQ + k * 16) * K::LDX + np * 16);
#pragma unroll
            for (int m = 0; m < K::MT; ++m) {
              mma_bf16(S[m][2 * np], a[m], b[0], b[1]);
              mma_bf16(S[m][2 * np + 1], a[m], b[2], b[3]);
            }
          }
        }
      }
    }
    if (c + 1 < nchunks) {
      if (sw == 0) scalars(c + 1);
      publish(c + 1);
    }
  }
#pragma unroll
  for (int m = 0; m < K::MT; ++m)
#pragma unroll
    for (int c = 0; c < K::NC; ++c)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = st_row + 128 * m + qr + 8 * (e >> 1), d = st_col + 8 * c + 2 * qt + (e & 1);
        if (n < N && d < ncols) sp[(size_t)d * N + n] = S[m][c][e];
      }
}

template <int NT, int DVB>
static int chunks_launch(const bf16* xbc, long long ldx, const float* dt, long long ldt, const float* dt_bias, const float* a_log,
                         const float* skip, const int* segs, int n_seg, float* state, float* y, int H, int G, int N, int dv,
                         cudaStream_t s) {
  static HkSmemCache cache;
  constexpr size_t smem = ChunkShape<NT, DVB>::SMEM;
  if (int e = hk_allow_smem(state_space_chunks_kernel<NT, DVB>, smem, cache)) return e;
  dim3 grid((unsigned)(n_seg * H), (unsigned)((dv + DVB - 1) / DVB));
  return hk_launch(state_space_chunks_kernel<NT, DVB>, grid, dim3(512), smem, s, xbc, ldx, dt, ldt, dt_bias, a_log, skip, segs, state, y, H,
                   G, N, dv);
}

// As hk_state_space_walk for bf16 rows, meant for segments of some length.  Refuses what the 16-byte copies cannot take (N,
// dv or ldx no multiple of 8, an unaligned xbc) and states of more than 256 numbers a column.
HK_API int hk_state_space_chunks(const void* xbc, long long ldx, const float* dt, long long ldt, const float* dt_bias,
                                 const float* a_log, const float* skip, const int* segs, int n_seg, int n_rows, float* state, float* y,
                                 int H, int G, int N, int dv, void* stream) {
  if (n_seg <= 0 || n_rows <= 0) return 0;
  if (H < 1 || G < 1 || H % G || N < 1 || N > 256 || (N & 7) || dv < 1 || (dv & 7) || (ldx & 7) || ((uintptr_t)xbc & 15)) return HK_ERR_UNSUPPORTED;
  if ((uintptr_t)y & 7) return HK_ERR_UNSUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
#define CHUNKS(NT, DVB) chunks_launch<NT, DVB>((const bf16*)xbc, ldx, dt, ldt, dt_bias, a_log, skip, segs, n_seg, state, y, H, G, N, dv, s)
  // 64 columns a block share the scores; 32 where that leaves SMs without a block
  const bool wide = dv > 32 && (long long)n_seg * H * ((dv + 63) / 64) * 4 >= 3 * 148;
  if (N <= 32) return wide ? CHUNKS(32, 64) : CHUNKS(32, 32);
  if (N <= 64) return wide ? CHUNKS(64, 64) : CHUNKS(64, 32);
  if (N <= 128) return wide ? CHUNKS(128, 64) : CHUNKS(128, 32);
  return CHUNKS(256, 16);
#undef CHUNKS
}

// ------------------------------------------------------------------ the gate, then a norm over equal parts of the row
// u = y silu(z); each of `parts` equal parts of a row over its own root mean square (eps inside the root), times the
// weight, narrowed to T.  A block per (token, part); the part's u stays in shared memory between the two passes.
template <typename T, int V>
__global__ void gated_part_norm_kernel(const float* __restrict__ y, const float* __restrict__ z, long long ldz,
                                       const float* __restrict__ weight, T* __restrict__ out, int W, int width, float eps) {
  extern __shared__ __align__(16) float u[];        // [width]
  __shared__ float warp_part[32];
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int p0 = blockIdx.y * width;
  const float* yr = y + t * W + p0;
  const float* zr = z + t * ldz + p0;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
    float yv[V], zv[V];
    if (V == 4) {
      *reinterpret_cast<float4*>(yv) = *reinterpret_cast<const float4*>(yr + i);
      *reinterpret_cast<float4*>(zv) = *reinterpret_cast<const float4*>(zr + i);
    } else {
      yv[0] = yr[i];
      zv[0] = zr[i];
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float g = yv[e] * (zv[e] / (1.0f + expf(-zv[e])));
      u[i + e] = g;
      ss = fmaf(g, g, ss);
    }
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) warp_part[threadIdx.x >> 5] = ss;
  __syncthreads();
  float total = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) total += warp_part[i];
  const float inv = 1.0f / sqrtf(total / (float)width + eps);
  T* o = out + t * W + p0;
  const float* wp = weight + p0;
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
    if (V == 4) {
      const float4 w4 = *reinterpret_cast<const float4*>(wp + i), u4 = *reinterpret_cast<const float4*>(u + i);
      const float r0 = u4.x * inv * w4.x, r1 = u4.y * inv * w4.y, r2 = u4.z * inv * w4.z, r3 = u4.w * inv * w4.w;
      if (sizeof(T) == 2) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(r0, r1), hi = __floats2bfloat162_rn(r2, r3);
        *reinterpret_cast<uint2*>(o + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
      } else {
        *reinterpret_cast<float4*>(o + i) = make_float4(r0, r1, r2, r3);
      }
    } else {
      o[i] = from_f32<T>(u[i] * inv * wp[i]);
    }
  }
}

template <typename T>
static int gated_part_norm(const float* y, const float* z, long long ldz, const float* weight, T* out, int n, int W, int parts, float eps,
                           cudaStream_t s) {
  const int width = W / parts;
  const bool vec = (width & 3) == 0 && (ldz & 3) == 0 &&
                   (((uintptr_t)y | (uintptr_t)z | (uintptr_t)weight | (uintptr_t)out) & 15) == 0;
  const int items = vec ? width / 4 : width;
  const int threads = items >= 256 ? 256 : items > 64 ? 128 : items > 32 ? 64 : 32;
  const size_t smem = (size_t)width * sizeof(float);
  dim3 grid((unsigned)n, (unsigned)parts);
  if (vec) {
    static HkSmemCache cache;
    if (int e = hk_allow_smem(gated_part_norm_kernel<T, 4>, smem, cache)) return e;
    return hk_launch_pdl(gated_part_norm_kernel<T, 4>, grid, dim3(threads), smem, s, y, z, ldz, weight, out, W, width, eps);
  }
  static HkSmemCache cache;
  if (int e = hk_allow_smem(gated_part_norm_kernel<T, 1>, smem, cache)) return e;
  return hk_launch_pdl(gated_part_norm_kernel<T, 1>, grid, dim3(threads), smem, s, y, z, ldz, weight, out, W, width, eps);
}

// y float32 [n, W], z a float32 column slice [n, W] (row stride ldz), weight float32 [W], out [n, W]; W a multiple of parts.
HK_API int hk_gated_part_norm(const float* y, const float* z, long long ldz, const float* weight, void* out, int out_dtype, int n, int W,
                              int parts, float eps, void* stream) {
  if (n <= 0) return 0;
  if (parts < 1 || W % parts || W / parts > 50 * 1024 || parts > 65535) return HK_ERR_UNSUPPORTED;
  if (out_dtype == HK_F32) return gated_part_norm<float>(y, z, ldz, weight, (float*)out, n, W, parts, eps, (cudaStream_t)stream);
  if (out_dtype == HK_BF16) return gated_part_norm<bf16>(y, z, ldz, weight, (bf16*)out, n, W, parts, eps, (cudaStream_t)stream);
  return HK_ERR_UNSUPPORTED;
}
