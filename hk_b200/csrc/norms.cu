// Row-wise norms beyond the plain RMS norm:
//   * layer norm: out = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b, the deviations squared (not the square of the
//     mean taken off the mean square), optionally over a list of rows;
//   * the end of a layer half whose two mixers stand side by side: both results over their own root mean square, times
//     their weights and factors, added onto the float32 residual stream, and, in the same pass over the row, the layer
//     norm that the next sublayer reads.
// All arithmetic is float32.  A row's sums run in a fixed order that its width alone decides (thread-strided partials,
// warp tree, then warps in order), so a row's result does not depend on what else is in the batch.
#include "common.cuh"

namespace {

constexpr int NT = 256, NW = NT / 32;

// The block's sum of `v` for every thread; `part` [NW] belongs to one call and is not written again before the next barrier
// behind it.
__device__ __forceinline__ float block_sum(float v, float* part) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float total = 0.f;
#pragma unroll
  for (int i = 0; i < NW; ++i) total += part[i];
  return total;
}

template <typename TO>
__device__ __forceinline__ void store4(TO* dst, float a, float b, float c, float d) {
  if (sizeof(TO) == 4) {
    *reinterpret_cast<float4*>(dst) = make_float4(a, b, c, d);
  } else {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
  }
}

// Layer norm of a row held as PER float4 a thread (chunk k * NT + thread; what lies past the row is zero).
template <typename TO, int PER>
__device__ __forceinline__ void layer_norm_row(const float4* v, const float* w, const float* b, TO* dst, int d, float eps,
                                               float* part0, float* part1) {
  const int chunks = d >> 2;
  float s = 0.f;
#pragma unroll
  for (int k = 0; k < PER; ++k) s += (v[k].x + v[k].y) + (v[k].z + v[k].w);
  const float mean = block_sum(s, part0) / (float)d;
  s = 0.f;
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    if (threadIdx.x + k * NT >= chunks) continue;
    const float a = v[k].x - mean, e = v[k].y - mean, f = v[k].z - mean, g = v[k].w - mean;
    s = fmaf(a, a, s);
    s = fmaf(e, e, s);
    s = fmaf(f, f, s);
    s = fmaf(g, g, s);
  }
  const float inv = 1.0f / sqrtf(block_sum(s, part1) / (float)d + eps);
  const float4* wv = reinterpret_cast<const float4*>(w);
  const float4* bv = reinterpret_cast<const float4*>(b);
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int c = threadIdx.x + k * NT;
    if (c >= chunks) continue;
    const float4 g = wv[c], h = bv[c];
    store4<TO>(dst + 4 * c, fmaf((v[k].x - mean) * inv, g.x, h.x), fmaf((v[k].y - mean) * inv, g.y, h.y),
               fmaf((v[k].z - mean) * inv, g.z, h.z), fmaf((v[k].w - mean) * inv, g.w, h.w));
  }
}

// Layer norm of a row of any width that every thread of the block can read; the values past the barriers are read again.
template <typename TO>
__device__ __forceinline__ void layer_norm_row_any(const float* src, const float* w, const float* b, TO* dst, int d, float eps,
                                                   float* part0, float* part1) {
  float s = 0.f;
  for (int i = threadIdx.x; i < d; i += NT) s += src[i];
  const float mean = block_sum(s, part0) / (float)d;
  s = 0.f;
  for (int i = threadIdx.x; i < d; i += NT) {
    const float a = src[i] - mean;
    s = fmaf(a, a, s);
  }
  const float inv = 1.0f / sqrtf(block_sum(s, part1) / (float)d + eps);
  for (int i = threadIdx.x; i < d; i += NT) dst[i] = from_f32<TO>(fmaf((src[i] - mean) * inv, w[i], b[i]));
}

}  // namespace

// ----------------------------------------------------------------------------- layer norm
template <typename TO, int PER>
__global__ void __launch_bounds__(NT)
layer_norm_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ b, const int* __restrict__ rows,
                  TO* __restrict__ out, int d, float eps) {
  __shared__ float part[2][NW];
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x;
  const float4* src = reinterpret_cast<const float4*>(x + (size_t)(rows ? rows[r] : r) * d);
  float4 v[PER];
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int c = threadIdx.x + k * NT;
    v[k] = c < (d >> 2) ? src[c] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  layer_norm_row<TO, PER>(v, w, b, out + (size_t)r * d, d, eps, part[0], part[1]);
}

template <typename TO>
__global__ void __launch_bounds__(NT)
layer_norm_any_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ b, const int* __restrict__ rows,
                      TO* __restrict__ out, int d, float eps) {
  __shared__ float part[2][NW];
  const int r = blockIdx.x;
  layer_norm_row_any<TO>(x + (size_t)(rows ? rows[r] : r) * d, w, b, out + (size_t)r * d, d, eps, part[0], part[1]);
}

template <typename TO>
static int layer_norm(const float* x, const float* w, const float* b, const int* rows, TO* out, int n, int d, float eps, cudaStream_t s) {
  const int chunks = d >> 2;
  if ((d & 3) == 0 && chunks <= 8 * NT && (((uintptr_t)x | (uintptr_t)w | (uintptr_t)b | (uintptr_t)out) & 15) == 0) {
    if (chunks <= NT) return hk_launch_pdl(layer_norm_kernel<TO, 1>, dim3(n), dim3(NT), 0, s, x, w, b, rows, out, d, eps);
    if (chunks <= 2 * NT) return hk_launch_pdl(layer_norm_kernel<TO, 2>, dim3(n), dim3(NT), 0, s, x, w, b, rows, out, d, eps);
    if (chunks <= 4 * NT) return hk_launch_pdl(layer_norm_kernel<TO, 4>, dim3(n), dim3(NT), 0, s, x, w, b, rows, out, d, eps);
    return hk_launch_pdl(layer_norm_kernel<TO, 8>, dim3(n), dim3(NT), 0, s, x, w, b, rows, out, d, eps);
  }
  return hk_launch(layer_norm_any_kernel<TO>, dim3(n), dim3(NT), 0, s, x, w, b, rows, out, d, eps);
}

// x float32 [*, d], w and b float32 [d], rows int32 [n_out] or null (row r of out is row r of x), out [n_out, d].
HK_API int hk_layer_norm(const float* x, const float* w, const float* b, const int* rows, void* out, int out_dtype, int n_out, int d,
                         float eps, void* stream) {
  if (n_out <= 0) return 0;
  if (d < 1) return HK_ERR_UNSUPPORTED;
  if (out_dtype == HK_F32) return layer_norm<float>(x, w, b, rows, (float*)out, n_out, d, eps, (cudaStream_t)stream);
  if (out_dtype == HK_BF16) return layer_norm<bf16>(x, w, b, rows, (bf16*)out, n_out, d, eps, (cudaStream_t)stream);
  return HK_ERR_UNSUPPORTED;
}

// ----------------------------------------------------------------------------- two normed results onto the residual
// residual[r] += ls * N(a[r] + a_bias) * wa + rs * N(b[r]) * wb with N(y) = y / sqrt(mean(y^2) + eps) over the row; a_bias
// (or null) is added before the norm.  `accumulate` 0 stores instead.  With `lw` (and lb, lout) the new residual row's layer
// norm goes to lout.
struct PairNorm {
  const float *a, *a_bias, *wa, *b, *wb;
  float eps_a, eps_b, ls, rs;
  float* residual;
  int accumulate;
  const float *lw, *lb;
  float leps;
};

template <typename TO, int PER>
__global__ void __launch_bounds__(NT) pair_norm_add_kernel(const PairNorm p, TO* __restrict__ lout, int d) {
  __shared__ float part[4][NW];
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = (size_t)blockIdx.x * d;
  const int chunks = d >> 2;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 a[PER], b[PER], r[PER];
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int c = threadIdx.x + k * NT;
    const bool in = c < chunks;
    a[k] = in ? reinterpret_cast<const float4*>(p.a + row)[c] : zero;
    b[k] = in ? reinterpret_cast<const float4*>(p.b + row)[c] : zero;
    r[k] = in && p.accumulate ? reinterpret_cast<const float4*>(p.residual + row)[c] : zero;
    if (in && p.a_bias) {
      const float4 e = reinterpret_cast<const float4*>(p.a_bias)[c];
      a[k] = make_float4(a[k].x + e.x, a[k].y + e.y, a[k].z + e.z, a[k].w + e.w);
    }
  }
  float sa = 0.f, sb = 0.f;
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    sa = fmaf(a[k].x, a[k].x, fmaf(a[k].y, a[k].y, fmaf(a[k].z, a[k].z, fmaf(a[k].w, a[k].w, sa))));
    sb = fmaf(b[k].x, b[k].x, fmaf(b[k].y, b[k].y, fmaf(b[k].z, b[k].z, fmaf(b[k].w, b[k].w, sb))));
  }
  const float ta = block_sum(sa, part[0]), tb = block_sum(sb, part[1]);
  const float ia = p.ls / sqrtf(ta / (float)d + p.eps_a), ib = p.rs / sqrtf(tb / (float)d + p.eps_b);
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int c = threadIdx.x + k * NT;
    if (c >= chunks) continue;
    const float4 u = reinterpret_cast<const float4*>(p.wa)[c], v = reinterpret_cast<const float4*>(p.wb)[c];
    r[k].x += fmaf(a[k].x * ia, u.x, b[k].x * ib * v.x);
    r[k].y += fmaf(a[k].y * ia, u.y, b[k].y * ib * v.y);
    r[k].z += fmaf(a[k].z * ia, u.z, b[k].z * ib * v.z);
    r[k].w += fmaf(a[k].w * ia, u.w, b[k].w * ib * v.w);
    reinterpret_cast<float4*>(p.residual + row)[c] = r[k];
  }
  if (lout) layer_norm_row<TO, PER>(r, p.lw, p.lb, lout + row, d, p.leps, part[2], part[3]);
}

template <typename TO>
__global__ void __launch_bounds__(NT) pair_norm_add_any_kernel(const PairNorm p, TO* __restrict__ lout, int d) {
  __shared__ float part[4][NW];
  const size_t row = (size_t)blockIdx.x * d;
  float sa = 0.f, sb = 0.f;
  for (int i = threadIdx.x; i < d; i += NT) {
    const float a = p.a[row + i] + (p.a_bias ? p.a_bias[i] : 0.f), b = p.b[row + i];
    sa = fmaf(a, a, sa);
    sb = fmaf(b, b, sb);
  }
  const float ta = block_sum(sa, part[0]), tb = block_sum(sb, part[1]);
  const float ia = p.ls / sqrtf(ta / (float)d + p.eps_a), ib = p.rs / sqrtf(tb / (float)d + p.eps_b);
  for (int i = threadIdx.x; i < d; i += NT) {
    const float a = p.a[row + i] + (p.a_bias ? p.a_bias[i] : 0.f);
    const float sum = fmaf(a * ia, p.wa[i], p.b[row + i] * ib * p.wb[i]);
    p.residual[row + i] = p.accumulate ? p.residual[row + i] + sum : sum;
  }
  if (!lout) return;
  layer_norm_row_any<TO>(p.residual + row, p.lw, p.lb, lout + row, d, p.leps, part[2], part[3]);   // a thread reads what it wrote itself
}

template <typename TO>
static int pair_norm_add(const PairNorm& p, TO* lout, int n, int d, cudaStream_t s) {
  const int chunks = d >> 2;
  const uintptr_t all = (uintptr_t)p.a | (uintptr_t)p.a_bias | (uintptr_t)p.wa | (uintptr_t)p.b | (uintptr_t)p.wb | (uintptr_t)p.residual |
                        (uintptr_t)p.lw | (uintptr_t)p.lb | (uintptr_t)lout;
  if ((d & 3) == 0 && chunks <= 8 * NT && (all & 15) == 0) {
    if (chunks <= NT) return hk_launch_pdl(pair_norm_add_kernel<TO, 1>, dim3(n), dim3(NT), 0, s, p, lout, d);
    if (chunks <= 2 * NT) return hk_launch_pdl(pair_norm_add_kernel<TO, 2>, dim3(n), dim3(NT), 0, s, p, lout, d);
    if (chunks <= 4 * NT) return hk_launch_pdl(pair_norm_add_kernel<TO, 4>, dim3(n), dim3(NT), 0, s, p, lout, d);
    return hk_launch_pdl(pair_norm_add_kernel<TO, 8>, dim3(n), dim3(NT), 0, s, p, lout, d);
  }
  return hk_launch(pair_norm_add_any_kernel<TO>, dim3(n), dim3(NT), 0, s, p, lout, d);
}

// a, b, residual float32 [n, d] (a and b not the residual); a_bias float32 [d] or null; wa, wb float32 [d]; lw, lb float32 [d]
// and lout [n, d], or all three null.
HK_API int hk_pair_norm_add(const float* a, const float* a_bias, const float* wa, float eps_a, float ls, const float* b, const float* wb,
                            float eps_b, float rs, float* residual, int accumulate, const float* lw, const float* lb, float leps,
                            void* lout, int lout_dtype, int n, int d, void* stream) {
  if (n <= 0) return 0;
  if (d < 1 || (lout && (!lw || !lb))) return HK_ERR_UNSUPPORTED;
  const PairNorm p = {a, a_bias, wa, b, wb, eps_a, eps_b, ls, rs, residual, accumulate, lw, lb, leps};
  if (lout_dtype == HK_F32) return pair_norm_add<float>(p, (float*)lout, n, d, (cudaStream_t)stream);
  if (lout_dtype == HK_BF16) return pair_norm_add<bf16>(p, (bf16*)lout, n, d, (cudaStream_t)stream);
  return HK_ERR_UNSUPPORTED;
}
