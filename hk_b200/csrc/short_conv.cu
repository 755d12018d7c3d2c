// The short causal convolution per channel that some mixers put behind their projections, with the request's last inputs
// kept in its state slot between steps (float32).
//
// A step's batch is described by a segment table int32 [n_seg, 3] = (state slot, first row, rows), as for the recurrent
// mixers' scans; an output depends on the inputs before it alone, never on the cut of the prompt, the batch or the slot.
#include "common.cuh"

// ------------------------------------------------------------------ short causal convolution per channel
// y[t, c] = act(bias[c] + sum_j w[c, j] * x[t - (taps - 1) + j, c]) over the rows of every segment, with act = silu (1) or
// the identity (0) and a bias or none: the last column of w is the current token's.  The sum and the activation are
// float32; y is float32 or the storage type.  The inputs before a segment's first row come from the request's tail
// (state [slots, taps - 1, C], the last taps - 1 inputs of the request, zero at its start), which the same call
// moves on.  x (float32) and y are column slices [n, C] of wider matrices.  A thread owns one channel of one chunk
// of a segment's tokens; the threads of the first chunk read the old tail before they write the new one, and
// nobody else touches it.
#define SC_TOKENS 32
#define SC_GROUP 8
#define SC_MAX_TAPS 16

// The thread walks its tokens in groups of SC_GROUP: the group's inputs are loaded at once (each input is read once; the
// taps - 1 before them stay in registers from the group before), then the group's outputs are summed, oldest tap first.
// A segment of one row (a decoded token) takes a path of its own with the same sum.  TAPS: the most taps an instance holds.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
short_conv_kernel(const float* __restrict__ x, long long ldx, const float* __restrict__ w, const float* __restrict__ bias,
                  const int* __restrict__ segs, float* __restrict__ tail, T* __restrict__ y, long long ldy, int C, int taps, int act) {
  const int seg = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  const int slot = segs[seg * 3], row0 = segs[seg * 3 + 1], count = segs[seg * 3 + 2];
  const int t0 = blockIdx.z * SC_TOKENS;
  if (c >= C || t0 >= count) return;
  const int back = taps - 1;
  float* tl = tail + (size_t)slot * back * C + c;
  auto input = [&](int r) -> float {            // the request's input r rows from the segment's first (r may be negative)
    return r >= 0 ? x[(size_t)(row0 + r) * ldx + c] : tl[(size_t)(back + r) * C];
  };
  float wr[TAPS];                               // wr[s]: the weight of the input s tokens back
  float hist[TAPS];                             // hist[s], s >= 1: the input s tokens before the group's first
  if (TAPS == 4 && taps == 4 && ((uintptr_t)w & 15) == 0) {
    const float4 q = *reinterpret_cast<const float4*>(w + (size_t)c * 4);
    wr[0] = q.w; wr[TAPS > 1 ? 1 : 0] = q.z; wr[TAPS > 2 ? 2 : 0] = q.y; wr[TAPS > 3 ? 3 : 0] = q.x;
  } else {
#pragma unroll
    for (int s = 0; s < TAPS; ++s) wr[s] = s <= back ? w[(size_t)c * taps + back - s] : 0.f;
  }
#pragma unroll
  for (int s = 0; s < TAPS; ++s) hist[s] = (s >= 1 && s <= back) ? input(t0 - s) : 0.f;
  const float first = bias != nullptr ? bias[c] : 0.f;
  if (count == 1) {
    const float now = x[(size_t)row0 * ldx + c];
    float acc = first;
#pragma unroll
    for (int s = TAPS - 1; s >= 1; --s)
      if (s <= back) acc = fmaf(wr[s], hist[s], acc);
    acc = fmaf(wr[0], now, acc);
    y[(size_t)row0 * ldy + c] = from_f32<T>(act ? acc / (1.0f + expf(-acc)) : acc);
#pragma unroll
    for (int s = TAPS - 1; s >= 2; --s)
      if (s <= back) tl[(size_t)(back - s) * C] = hist[s - 1];
    if (back > 0) tl[(size_t)(back - 1) * C] = now;
    return;
  }
  const int t1 = min(count, t0 + SC_TOKENS);
  for (int tg = t0; tg < t1; tg += SC_GROUP) {
    float nw[SC_GROUP];
#pragma unroll
    for (int u = 0; u < SC_GROUP; ++u) nw[u] = tg + u < t1 ? x[(size_t)(row0 + tg + u) * ldx + c] : 0.f;
    float acc[SC_GROUP];
#pragma unroll
    for (int u = 0; u < SC_GROUP; ++u) acc[u] = first;
#pragma unroll
    for (int s = TAPS - 1; s >= 0; --s) {
      if (s <= back) {
#pragma unroll
        for (int u = 0; u < SC_GROUP; ++u) acc[u] = fmaf(wr[s], u >= s ? nw[u >= s ? u - s : 0] : hist[u >= s ? 0 : s - u], acc[u]);
      }
    }
#pragma unroll
    for (int u = 0; u < SC_GROUP; ++u)
      if (tg + u < t1) y[(size_t)(row0 + tg + u) * ldy + c] = from_f32<T>(act ? acc[u] / (1.0f + expf(-acc[u])) : acc[u]);
    float next[TAPS];
#pragma unroll
    for (int s = 1; s < TAPS; ++s) next[s] = s <= SC_GROUP ? nw[s <= SC_GROUP ? SC_GROUP - s : 0] : hist[s <= SC_GROUP ? 0 : s - SC_GROUP];
#pragma unroll
    for (int s = 1; s < TAPS; ++s) hist[s] = next[s];
  }
  if (blockIdx.z == 0 && back > 0) {
    float keep[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
      if (j < back) keep[j] = input(count - back + j);
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
      if (j < back) tl[(size_t)j * C] = keep[j];
  }
}

template <typename T, int TAPS>
static int short_conv(const float* x, long long ldx, const float* w, const float* bias, const int* segs, int n_seg, int n_rows, float* tail,
                      T* y, long long ldy, int C, int taps, int act, cudaStream_t s) {
  // a step of single rows needs no second block of tokens; else as many as the longest segment may have
  const int longest = n_rows - n_seg + 1;
  dim3 grid((unsigned)n_seg, (unsigned)((C + 127) / 128), (unsigned)((longest + SC_TOKENS - 1) / SC_TOKENS));
  return hk_launch(short_conv_kernel<T, TAPS>, grid, dim3(128), 0, s, x, ldx, w, bias, segs, tail, y, ldy, C, taps, act);
}

HK_API int hk_short_conv(const float* x, long long ldx, const float* w, const float* bias, const int* segs, int n_seg, int n_rows,
                         float* tail, void* y, int y_dtype, long long ldy, int C, int taps, int act, void* stream) {
  if (n_seg <= 0 || n_rows <= 0 || C <= 0) return 0;
  if (taps < 1 || taps > SC_MAX_TAPS || act < 0 || act > 1 || n_rows < n_seg) return HK_ERR_UNSUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
#define SHORT_CONV(T)                                                                                                     \
  (taps <= 4 ? short_conv<T, 4>(x, ldx, w, bias, segs, n_seg, n_rows, tail, (T*)y, ldy, C, taps, act, s)                  \
             : short_conv<T, SC_MAX_TAPS>(x, ldx, w, bias, segs, n_seg, n_rows, tail, (T*)y, ldy, C, taps, act, s))
  if (y_dtype == HK_F32) return SHORT_CONV(float);
  if (y_dtype == HK_BF16) return SHORT_CONV(bf16);
  return HK_ERR_UNSUPPORTED;
#undef SHORT_CONV
}
