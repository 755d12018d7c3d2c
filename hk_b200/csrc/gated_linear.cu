// Linear attention with a decay per key channel (gated linear attention): the recurrence over the rows of every request of
// a step, its state kept in float32 in the request's state slot between steps.
//
// Per head a matrix state S [dk, dv] (zero at a request's start):
//     S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T (q_scale q_t),   alpha_t = sigmoid(z_t)^(1 / tau) per key channel
// with the logits z = W2 (W1 h) + b of a low-rank projection whose second factor is applied here, in float32.  A step's batch
// is described by a segment table int32 [n_seg, 3] = (state slot, first row, rows).  q, k and v are float32 column slices of
// a projection's output.  The state of a slot is stored [H, dv, dk]: a column's dk entries are neighbours, so the lanes that
// share a column read and write whole lines.
#include "common.cuh"

namespace {

__device__ __forceinline__ float logsigmoid_f(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

template <int BYTES>
__device__ __forceinline__ void cp_async(void* dst, const void* src) {
  if (BYTES == 16)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
  else
    asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "n"(BYTES) : "memory");
}

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

}  // namespace

// ------------------------------------------------------------------ the decays
// la[t, c] = log2(alpha) = logsigmoid(sum_r w2[c, r] hid[t, r] + bias[c]) / tau * log2(e).  A thread owns one channel and
// TT tokens, so a channel's row of w2 is read once per TT tokens; the tokens' hidden values come through shared memory.
template <int TT>
__global__ void __launch_bounds__(128)
gla_decay_kernel(const float* __restrict__ hid, long long ldh, int R, const float* __restrict__ w2, const float* __restrict__ bias,
                 float* __restrict__ la, int n, int K, float factor) {
  extern __shared__ float hs[];                    // [R][TT]
  pdl_launch_dependents();
  const int c = blockIdx.y * 128 + threadIdx.x, t0 = blockIdx.x * TT;
  pdl_wait();
  for (int i = threadIdx.x; i < R * TT; i += 128) {
    const int t = t0 + i / R;
    hs[(i % R) * TT + i / R] = t < n ? hid[(size_t)t * ldh + i % R] : 0.f;
  }
  __syncthreads();
  if (c >= K) return;
  float acc[TT];
#pragma unroll
  for (int t = 0; t < TT; ++t) acc[t] = 0.f;
  const float* wr = w2 + (size_t)c * R;
  int r = 0;
  if ((R & 3) == 0 && ((uintptr_t)w2 & 15) == 0) {
    for (; r < R; r += 4) {
      const float4 w = *reinterpret_cast<const float4*>(wr + r);
#pragma unroll
      for (int t = 0; t < TT; ++t) {
        acc[t] = fmaf(w.x, hs[r * TT + t], acc[t]);
        acc[t] = fmaf(w.y, hs[(r + 1) * TT + t], acc[t]);
        acc[t] = fmaf(w.z, hs[(r + 2) * TT + t], acc[t]);
        acc[t] = fmaf(w.w, hs[(r + 3) * TT + t], acc[t]);
      }
    }
  }
  for (; r < R; ++r) {
    const float w = wr[r];
#pragma unroll
    for (int t = 0; t < TT; ++t) acc[t] = fmaf(w, hs[r * TT + t], acc[t]);
  }
  const float b = bias[c];
#pragma unroll
  for (int t = 0; t < TT; ++t)
    if (t0 + t < n) la[(size_t)(t0 + t) * K + c] = logsigmoid_f(acc[t] + b) * factor;
}

// hid float32 [n, R] (row stride ldh), w2 float32 [K, R], bias float32 [K], la float32 [n, K].
HK_API int hk_gla_decay(const float* hid, long long ldh, int R, const float* w2, const float* bias, float* la, int n, int K, float tau,
                        void* stream) {
  if (n <= 0) return 0;
  if (R < 1 || R > 1024 || K < 1 || !(tau > 0.f)) return HK_ERR_UNSUPPORTED;
  const float factor = 1.4426950408889634f / tau;
  cudaStream_t s = (cudaStream_t)stream;
  if ((long long)n * K >= 8ll * 128 * 148)
    return hk_launch_pdl(gla_decay_kernel<8>, dim3((unsigned)((n + 7) / 8), (unsigned)((K + 127) / 128)), dim3(128), (size_t)R * 8 * sizeof(float), s,
                         hid, ldh, R, w2, bias, la, n, K, factor);
  return hk_launch_pdl(gla_decay_kernel<1>, dim3((unsigned)n, (unsigned)((K + 127) / 128)), dim3(128), (size_t)R * sizeof(float), s, hid, ldh, R,
                       w2, bias, la, n, K, factor);
}

// ------------------------------------------------------------------ the walk, token by token
// A block of 128 threads owns `cols` = 128 / L * CPT columns of one head's state for one segment.  A column's entries are
// spread over L lanes, RPT per lane, in registers: lane `sub` holds the entries 4 (q L + sub) .. + 3 for q < RPT / 4, and a
// lane group holds CPT columns (they share every load of a token's vectors).  Rows arrive in chunks of `chunk` tokens through
// a two-stage cp.async ring; a chunk's log decays become decays once, in place.  The chain that the next token waits for is
// one multiply and one fused multiply-add per state entry; the read-out's sums over the L lanes hang off it.
template <int L, int RPT, int CPT>
__global__ void __launch_bounds__(128)
gla_walk_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v, long long ld,
                const float* __restrict__ la, const int* __restrict__ segs, float* __restrict__ state, float* __restrict__ out,
                long long ldo, int H, int dk, int dv, float q_scale, int chunk, int vec) {
  constexpr int P = L * RPT;
  constexpr int COLS = 128 / L * CPT;
  constexpr int R = 3 * P + COLS;                  // floats of a token in a stage: q, k, decay, the block's values
  extern __shared__ __align__(16) float rows[];    // [2][chunk][R]
  const int seg = blockIdx.x / H, h = blockIdx.x % H;
  const int slot = segs[seg * 3], row0 = segs[seg * 3 + 1], count = segs[seg * 3 + 2];
  const int col0 = blockIdx.y * COLS, ncols = min(COLS, dv - col0);
  const int tid = threadIdx.x, sub = tid % L, c0 = (tid / L) * CPT;

  float S[CPT][RPT];
  float* sp = state + (((size_t)slot * H + h) * dv + col0 + c0) * dk;
  const bool whole = (dk & 3) == 0;
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int e = 0; e < RPT / 4; ++e) {
      const int i = 4 * (e * L + sub);
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c0 + c < ncols) {
        const float* p = sp + (size_t)c * dk + i;
        if (whole) {
          if (i < dk) x = *reinterpret_cast<const float4*>(p);
        } else {
          if (i < dk) x.x = p[0];
          if (i + 1 < dk) x.y = p[1];
          if (i + 2 < dk) x.z = p[2];
          if (i + 3 < dk) x.w = p[3];
        }
      }
      S[c][4 * e] = x.x; S[c][4 * e + 1] = x.y; S[c][4 * e + 2] = x.z; S[c][4 * e + 3] = x.w;
    }
  if (dk < P || ncols < COLS) {                    // what no copy below ever touches: the padding must not hold NaN patterns
    for (int i = tid; i < 2 * chunk * R; i += 128) rows[i] = 0.f;
    __syncthreads();
  }

  const float* qs = q + (size_t)row0 * ld + (size_t)h * dk;
  const float* ks = k + (size_t)row0 * ld + (size_t)h * dk;
  const float* vs = v + (size_t)row0 * ld + (size_t)h * dv + col0;
  const size_t lda = (size_t)H * dk;
  const float* as = la + (size_t)row0 * lda + (size_t)h * dk;
  auto fetch = [&](int c) {                        // chunk c -> stage c & 1
    const int t0 = c * chunk, tc = min(chunk, count - t0);
    float* dst = rows + (size_t)(c & 1) * chunk * R;
    if (vec) {
      const int nb = dk / 4, nx = ncols / 4, per = 3 * nb + nx;
      for (int i = tid; i < tc * per; i += 128) {
        const int t = i / per, p = i - t * per;
        const size_t src = (size_t)(t0 + t) * ld;
        float* d = dst + (size_t)t * R;
        if (p < nb) cp_async<16>(d + p * 4, qs + src + p * 4);
        else if (p < 2 * nb) cp_async<16>(d + P + (p - nb) * 4, ks + src + (p - nb) * 4);
        else if (p < 3 * nb) cp_async<16>(d + 2 * P + (p - 2 * nb) * 4, as + (size_t)(t0 + t) * lda + (p - 2 * nb) * 4);
        else cp_async<16>(d + 3 * P + (p - 3 * nb) * 4, vs + src + (p - 3 * nb) * 4);
      }
    } else {
      const int per = 3 * dk + ncols;
      for (int i = tid; i < tc * per; i += 128) {
        const int t = i / per, p = i - t * per;
        const size_t src = (size_t)(t0 + t) * ld;
        float* d = dst + (size_t)t * R;
        if (p < dk) cp_async<4>(d + p, qs + src + p);
        else if (p < 2 * dk) cp_async<4>(d + P + p - dk, ks + src + p - dk);
        else if (p < 3 * dk) cp_async<4>(d + 2 * P + p - 2 * dk, as + (size_t)(t0 + t) * lda + p - 2 * dk);
        else cp_async<4>(d + 3 * P + p - 3 * dk, vs + src + p - 3 * dk);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int nchunks = (count + chunk - 1) / chunk;
  float* op = out + (size_t)row0 * ldo + (size_t)h * dv + col0 + c0;
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
    float* buf = rows + (size_t)(c & 1) * chunk * R;
    for (int i = tid; i < tc * P; i += 128)
      if (i % P < dk) {                            // (the padding stays 0: nothing brings it again)
        float* a = buf + (size_t)(i / P) * R + 2 * P + i % P;
        *a = exp2f(*a);
      }
    __syncthreads();
#pragma unroll 2
    for (int t = 0; t < tc; ++t) {
      const float* tok = buf + (size_t)t * R;
      float x[CPT], acc[CPT];
#pragma unroll
      for (int cc = 0; cc < CPT; ++cc) {
        x[cc] = tok[3 * P + c0 + cc];
        acc[cc] = 0.f;
      }
#pragma unroll
      for (int e = 0; e < RPT / 4; ++e) {
        const float4 r = *reinterpret_cast<const float4*>(tok + 4 * (e * L + sub));
        const float4 b = *reinterpret_cast<const float4*>(tok + P + 4 * (e * L + sub));
        const float4 a = *reinterpret_cast<const float4*>(tok + 2 * P + 4 * (e * L + sub));
#pragma unroll
        for (int cc = 0; cc < CPT; ++cc) {
          float* s = S[cc] + 4 * e;
          s[0] = fmaf(b.x, x[cc], a.x * s[0]);
          s[1] = fmaf(b.y, x[cc], a.y * s[1]);
          s[2] = fmaf(b.z, x[cc], a.z * s[2]);
          s[3] = fmaf(b.w, x[cc], a.w * s[3]);
          acc[cc] = fmaf(r.x, s[0], acc[cc]);
          acc[cc] = fmaf(r.y, s[1], acc[cc]);
          acc[cc] = fmaf(r.z, s[2], acc[cc]);
          acc[cc] = fmaf(r.w, s[3], acc[cc]);
        }
      }
      const int mine = sum_over_lanes<L, CPT>(acc, sub);
      if (writes_sum<L, CPT>(sub) && c0 + mine < ncols) op[(size_t)t * ldo + mine] = acc[0] * q_scale;
    }
    op += (size_t)tc * ldo;
    __syncthreads();                               // the stage may be filled again
  }
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int e = 0; e < RPT / 4; ++e) {
      const int i = 4 * (e * L + sub);
      if (c0 + c < ncols) {
        float* p = sp + (size_t)c * dk + i;
        if (whole) {
          if (i < dk) *reinterpret_cast<float4*>(p) = make_float4(S[c][4 * e], S[c][4 * e + 1], S[c][4 * e + 2], S[c][4 * e + 3]);
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (i + j < dk) p[j] = S[c][4 * e + j];
        }
      }
    }
}

// A step of single tokens (a decode step): the same arithmetic on one row per segment, without the ring and its barriers:
// everything a thread needs is asked for at once, straight into registers.  dk is a multiple of 4, and so are the distances
// of the rows.
template <int L, int RPT, int CPT>
__global__ void __launch_bounds__(128)
gla_step_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v, long long ld,
                const float* __restrict__ la, const int* __restrict__ segs, float* __restrict__ state, float* __restrict__ out,
                long long ldo, int H, int dk, int dv, float q_scale) {
  constexpr int COLS = 128 / L * CPT;
  const int seg = blockIdx.x / H, h = blockIdx.x % H;
  pdl_launch_dependents();
  const int slot = segs[seg * 3], row = segs[seg * 3 + 1];
  const int tid = threadIdx.x, sub = tid % L, c0 = blockIdx.y * COLS + (tid / L) * CPT;
  pdl_wait();
  float* sp = state + (((size_t)slot * H + h) * dv + c0) * dk;
  const float4* qs = reinterpret_cast<const float4*>(q + (size_t)row * ld + (size_t)h * dk);
  const float4* ks = reinterpret_cast<const float4*>(k + (size_t)row * ld + (size_t)h * dk);
  const float4* as = reinterpret_cast<const float4*>(la + ((size_t)row * H + h) * dk);
  const float* vs = v + (size_t)row * ld + (size_t)h * dv + c0;
  float4 S[CPT][RPT / 4], r[RPT / 4], b[RPT / 4], a[RPT / 4];
  float x[CPT], acc[CPT];
  bool in[RPT / 4];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int e = 0; e < RPT / 4; ++e) {
    const int i = e * L + sub;
    in[e] = 4 * i < dk;
#pragma unroll
    for (int c = 0; c < CPT; ++c) S[c][e] = in[e] && c0 + c < dv ? *reinterpret_cast<const float4*>(sp + (size_t)c * dk + 4 * i) : zero;
    r[e] = in[e] ? qs[i] : zero;
    b[e] = in[e] ? ks[i] : zero;
    a[e] = in[e] ? as[i] : zero;
  }
#pragma unroll
  for (int c = 0; c < CPT; ++c) {
    x[c] = c0 + c < dv ? vs[c] : 0.f;
    acc[c] = 0.f;
  }
#pragma unroll
  for (int e = 0; e < RPT / 4; ++e) {
    a[e] = make_float4(exp2f(a[e].x), exp2f(a[e].y), exp2f(a[e].z), exp2f(a[e].w));
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
      float4& s = S[c][e];
      s.x = fmaf(b[e].x, x[c], a[e].x * s.x);
      s.y = fmaf(b[e].y, x[c], a[e].y * s.y);
      s.z = fmaf(b[e].z, x[c], a[e].z * s.z);
      s.w = fmaf(b[e].w, x[c], a[e].w * s.w);
      acc[c] = fmaf(r[e].x, s.x, acc[c]);
      acc[c] = fmaf(r[e].y, s.y, acc[c]);
      acc[c] = fmaf(r[e].z, s.z, acc[c]);
      acc[c] = fmaf(r[e].w, s.w, acc[c]);
      if (in[e] && c0 + c < dv) *reinterpret_cast<float4*>(sp + (size_t)c * dk + 4 * (e * L + sub)) = s;
    }
  }
  const int mine = sum_over_lanes<L, CPT>(acc, sub);
  if (writes_sum<L, CPT>(sub) && c0 + mine < dv) out[(size_t)row * ldo + (size_t)h * dv + c0 + mine] = acc[0] * q_scale;
}

template <int L, int RPT, int CPT>
static int walk_launch(const float* q, const float* k, const float* v, long long ld, const float* la, const int* segs, int n_seg,
                       float* state, float* out, int H, int dk, int dv, float q_scale, int single, cudaStream_t s) {
  constexpr int COLS = 128 / L * CPT, R = 3 * L * RPT + COLS;
  const long long ldo = (long long)H * dv;
  dim3 grid((unsigned)(n_seg * H), (unsigned)((dv + COLS - 1) / COLS));
  const bool rows16 = (((uintptr_t)q | (uintptr_t)k | (uintptr_t)la) & 15) == 0 && (ld & 3) == 0 && (dk & 3) == 0;
  if (single && rows16)
    return hk_launch_pdl(gla_step_kernel<L, RPT, CPT>, grid, dim3(128), 0, s, q, k, v, ld, la, segs, state, out, ldo, H, dk, dv, q_scale);
  const int vec = rows16 && ((uintptr_t)v & 15) == 0 && (dv & 3) == 0 && COLS % 4 == 0;
  int chunk = 16;
  while (chunk > 2 && (size_t)2 * chunk * R * sizeof(float) > 48 * 1024) chunk >>= 1;
  const size_t smem = (size_t)2 * chunk * R * sizeof(float);
  static HkSmemCache cache;
  if (int e = hk_allow_smem(gla_walk_kernel<L, RPT, CPT>, smem, cache)) return e;
  return hk_launch(gla_walk_kernel<L, RPT, CPT>, grid, dim3(128), smem, s, q, k, v, ld, la, segs, state, out, ldo, H, dk, dv, q_scale,
                   chunk, vec);
}

// q, k [n, H dk] and v [n, H dv]: column slices of one float32 matrix (row stride ld); la float32 [n, H dk] (log2 of the
// decays); state float32 [slots, H, dv, dk]; out float32 [n, H dv].  single = 1 says that every segment has one row.  Four
// columns a lane group where the blocks fill the SMs twice, two where they do not (the layout of the sums does not depend on
// it).
HK_API int hk_gla_walk(const float* q, const float* k, const float* v, long long ld, const float* la, const int* segs, int n_seg,
                       float* state, float* out, int H, int dk, int dv, float q_scale, int single, void* stream) {
  if (n_seg <= 0) return 0;
  if (H < 1 || dk < 1 || dk > 1024 || dv < 1 || ((uintptr_t)state & 15)) return HK_ERR_UNSUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
#define WALK(L, RPT, CPT) walk_launch<L, RPT, CPT>(q, k, v, ld, la, segs, n_seg, state, out, H, dk, dv, q_scale, single, s)
#define WALK_ANY(L, RPT)                                                                                 \
  do {                                                                                                   \
    const bool many = (long long)n_seg * H * ((dv + 128 / L * 4 - 1) / (128 / L * 4)) >= 2 * 148;        \
    return many ? WALK(L, RPT, 4) : WALK(L, RPT, 2);                                                     \
  } while (0)
  if (dk <= 32) WALK_ANY(8, 4);
  if (dk <= 64) WALK_ANY(8, 8);
  if (dk <= 128) WALK_ANY(16, 8);
  if (dk <= 256) WALK_ANY(32, 8);
  if (dk <= 512) return WALK(32, 16, 2);
  return WALK(32, 32, 2);
#undef WALK_ANY
#undef WALK
}
