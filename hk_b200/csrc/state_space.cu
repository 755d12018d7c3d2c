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
      // the sum over the lanes: while a lane carries several columns, half of them go to the partner
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
      const int low = at;                          // the lanes below 2 * low now carry the same column
#pragma unroll
      for (int o = L / 2 / CPT; o > 0; o >>= 1) acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], o);
      float xm = x[0];
#pragma unroll
      for (int k = 1; k < CPT; ++k) xm = mine == k ? x[k] : xm;
      if ((low == 0 || (sub & (2 * low - 1)) == 0) && c0 + mine < ncols) yp[(size_t)t * ystep + mine] = fmaf(dskip, xm, acc[0]);
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

template <typename T, int L, int RPT, int CPT>
static int walk_launch(const T* xbc, long long ldx, const float* dt, long long ldt, const float* dt_bias, const float* a_log,
                       const float* skip, const int* segs, int n_seg, float* state, float* y, int H, int G, int N, int dv,
                       cudaStream_t s) {
  constexpr int COLS = 128 / L * CPT, R = 2 * L * RPT + COLS;
  constexpr int V = 16 / sizeof(T);
  const int inner = H * dv;
  const int vec = ((uintptr_t)xbc & 15) == 0 && ldx % V == 0 && inner % V == 0 && N % V == 0 && dv % V == 0 && COLS % V == 0;
  int chunk = 16;
  auto bytes = [&](int c) { return (size_t)2 * c * R * sizeof(T) + 2 * c * sizeof(float) + c * sizeof(float2); };
  while (chunk > 2 && bytes(chunk) > 48 * 1024) chunk >>= 1;
  const size_t smem = bytes(chunk);
  static HkSmemCache cache;
  if (int e = hk_allow_smem(state_space_walk_kernel<T, L, RPT, CPT>, smem, cache)) return e;
  dim3 grid((unsigned)(n_seg * H), (unsigned)((dv + COLS - 1) / COLS));
  return hk_launch(state_space_walk_kernel<T, L, RPT, CPT>, grid, dim3(128), smem, s, xbc, ldx, dt, ldt, dt_bias, a_log, skip, segs,
                   state, y, H, G, N, dv, chunk, vec);
}

// Four columns a lane group where the blocks fill the SMs twice, two where they do not (a column's entries spread over L
// lanes either way): the layout of the sums does not depend on it.
template <typename T>
static int walk(const T* xbc, long long ldx, const float* dt, long long ldt, const float* dt_bias, const float* a_log,
                const float* skip, const int* segs, int n_seg, float* state, float* y, int H, int G, int N, int dv, cudaStream_t s) {
#define WALK(L, RPT, CPT) walk_launch<T, L, RPT, CPT>(xbc, ldx, dt, ldt, dt_bias, a_log, skip, segs, n_seg, state, y, H, G, N, dv, s)
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
// [H]; state float32 [slots, H, dv, N]; y float32 [n, H dv].
HK_API int hk_state_space_walk(const void* xbc, int dtype, long long ldx, const float* dt, long long ldt, const float* dt_bias,
                               const float* a_log, const float* skip, const int* segs, int n_seg, int n_rows, float* state, float* y,
                               int H, int G, int N, int dv, void* stream) {
  if (n_seg <= 0 || n_rows <= 0) return 0;
  if (H < 1 || G < 1 || H % G || N < 1 || N > 1024 || dv < 1 || ((uintptr_t)state & 15)) return HK_ERR_UNSUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == HK_F32)
    return walk<float>((const float*)xbc, ldx, dt, ldt, dt_bias, a_log, skip, segs, n_seg, state, y, H, G, N, dv, s);
  if (dtype == HK_BF16)
    return walk<bf16>((const bf16*)xbc, ldx, dt, ldt, dt_bias, a_log, skip, segs, n_seg, state, y, H, G, N, dv, s);
  return HK_ERR_UNSUPPORTED;
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
