// Linear attention with a decay per key channel, prompt portions: the recurrence of gated_linear.cu,
//     S_t = diag(2^(la_t)) S_(t-1) + k_t v_t^T,   o_t = S_t^T (q_scale q_t),
// as matrix products over chunks of 64 tokens, all chunks of a step side by side.  With the chunk's cumulative log decays b_t
// (b of its first token that token's own) and its start state S_0, in exact arithmetic
//     o_t = (q_t 2^(b_t))^T S_0 + sum_(s <= t) A_ts v_s,      A_ts = sum_i q_t[i] k_s[i] 2^(b_t[i] - b_s[i])
//     S   = diag(2^(b_last)) S_0 + U,                         U = sum_s (k_s 2^(b_last - b_s)) v_s^T
//   1. states:  a block per (chunk, head, 64 or 128 value columns) makes U and the chunk's decay 2^(b_last);
//   2. carry:   a thread per four state entries walks a request's chunks, leaves every chunk's start state where its U was
//               and the request's last state in its slot;
//   3. outputs: a block per (chunk, head, 64 or 128 value columns) makes A and o.
// No exponent is ever positive, whatever the decays are: A's blocks of 16 x 16 tokens on the diagonal take 2^(b_t - b_s) entry
// by entry; a block below it takes the decays up to and from the boundary b_r before the rows' first token, q 2^(b_t - b_r)
// and k 2^(b_r - b_s).
//
// Scores, decays, cumulative sums and states are float32.  The products with v and with S_0 run on mma.sync: v is rounded to
// bf16 (it is a projection's output), and every float32 factor (decayed keys and queries, scores, the start state) is cut into
// three bf16 numbers whose sum is the float32 number to its last bit or two, with float32 sums; of the nine products of two
// such factors the six of the largest pieces are taken.
#include "common.cuh"

namespace {

constexpr int CQ = 64;          // tokens of a chunk
constexpr int SB = 16;          // tokens of a block of the scores
constexpr int NTH = 256;        // threads, eight warps

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
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
__device__ __forceinline__ uint32_t pack(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
// two float32 numbers as three pairs of bf16 whose sums they are
__device__ __forceinline__ void split3(float a, float b, uint32_t* out) {
#pragma unroll
  for (int p = 0; p < 3; ++p) {
    out[p] = pack(a, b);
    a -= __uint_as_float(out[p] << 16);
    b -= __uint_as_float(out[p] & 0xffff0000u);
  }
}

// A chunk as the host lists it.
struct Chunk {
  int row0, count;          // its rows of the step
};
// A request that is walked in chunks.
struct Request {
  int slot, chunk0, chunks;
};

// The chunk's log decays, rows [CQ][LD] of shared memory that hold la, become cumulative sums.  A thread takes 16 rows of a
// channel; `tot` [CQ / SB][NT] holds the blocks' sums.  Rows past the chunk's end hold 0.
template <int NT, int LD>
__device__ __forceinline__ void cumulate(float* b, float* tot) {
  for (int e = threadIdx.x; e < NT * (CQ / SB); e += NTH) {
    const int i = e % NT, blk = e / NT;
    float run = 0.f;
#pragma unroll
    for (int t = 0; t < SB; ++t) {
      float* p = b + (size_t)(blk * SB + t) * LD + i;
      run += *p;
      *p = run;
    }
    tot[e] = run;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < NT * (CQ / SB); e += NTH) {
    const int i = e % NT, blk = e / NT;
    float before = 0.f;
    for (int j = 0; j < blk; ++j) before += tot[j * NT + i];
    if (blk > 0) {
#pragma unroll
      for (int t = 0; t < SB; ++t) b[(size_t)(blk * SB + t) * LD + i] += before;
    }
  }
  __syncthreads();
}

}  // namespace

// ------------------------------------------------------------------ 1. states
// U [dv, dk] of a chunk and head: M = value columns, N = key channels, K = tokens.  Eight warps: a warp owns 16 value columns
// (and half of the channels where the block has 64 columns).
template <int NT, int DVB>
struct StatesShape {
  static constexpr int LB = NT + 4, LK = NT + 8, LV = DVB + 8;
  static constexpr int MT = DVB / 16, SPLIT = 8 / MT, NW = NT / 8 / SPLIT;      // channel tiles of 8 a warp
  static constexpr size_t SMEM = (size_t)CQ * LB * 4 + (size_t)(CQ / SB) * NT * 4 + ((size_t)3 * CQ * LK + (size_t)CQ * LV) * 2;
};

template <int NT, int DVB>
__global__ void __launch_bounds__(NTH)
gla_states_kernel(const float* __restrict__ k, const float* __restrict__ v, long long ld, const float* __restrict__ la,
                  const Chunk* __restrict__ chunks, float* __restrict__ u, float* __restrict__ decay, int H, int dk, int dv) {
  using K = StatesShape<NT, DVB>;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  float* b = reinterpret_cast<float*>(smem_raw);           // [CQ][LB]
  float* tot = b + CQ * K::LB;                             // [CQ / SB][NT]
  bf16* kw = reinterpret_cast<bf16*>(tot + (CQ / SB) * NT);     // [3][CQ][LK]
  bf16* vs = kw + 3 * CQ * K::LK;                          // [CQ][LV]
  const int c = blockIdx.x / H, h = blockIdx.x % H;
  const Chunk ch = chunks[c];
  const int col0 = blockIdx.y * DVB, ncols = min(DVB, dv - col0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  // everything is asked for at once; the keys wait in registers for the cumulative decays
  constexpr int NK = CQ * (NT / 4) / NTH, NV = CQ * (DVB / 4) / NTH;
  float4 kr[NK], lr[NK], vr[NV];
#pragma unroll
  for (int j = 0; j < NK; ++j) {
    const int e = tid + j * NTH, t = e / (NT / 4), i = (e % (NT / 4)) * 4;
    const bool in = t < ch.count && i < dk;
    lr[j] = in ? *reinterpret_cast<const float4*>(la + ((size_t)(ch.row0 + t) * H + h) * dk + i) : zero;
    kr[j] = in ? *reinterpret_cast<const float4*>(k + (size_t)(ch.row0 + t) * ld + (size_t)h * dk + i) : zero;
  }
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int e = tid + j * NTH, t = e / (DVB / 4), d = (e % (DVB / 4)) * 4;
    vr[j] = t < ch.count && d < ncols ? *reinterpret_cast<const float4*>(v + (size_t)(ch.row0 + t) * ld + (size_t)h * dv + col0 + d) : zero;
  }
#pragma unroll
  for (int j = 0; j < NK; ++j) {
    const int e = tid + j * NTH;
    *reinterpret_cast<float4*>(b + (e / (NT / 4)) * K::LB + (e % (NT / 4)) * 4) = lr[j];
  }
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int e = tid + j * NTH;
    *reinterpret_cast<uint2*>(vs + (e / (DVB / 4)) * K::LV + (e % (DVB / 4)) * 4) = make_uint2(pack(vr[j].x, vr[j].y), pack(vr[j].z, vr[j].w));
  }
  __syncthreads();
  cumulate<NT, K::LB>(b, tot);
  const float* last = b + (CQ - 1) * K::LB;
  if (blockIdx.y == 0)
    for (int i = tid; i < dk; i += NTH) decay[((size_t)c * H + h) * dk + i] = exp2_f(last[i]);
#pragma unroll
  for (int j = 0; j < NK; ++j) {
    const int e = tid + j * NTH, t = e / (NT / 4), i = (e % (NT / 4)) * 4;
    const float4 x0 = kr[j], z = *reinterpret_cast<const float4*>(last + i), y = *reinterpret_cast<const float4*>(b + t * K::LB + i);
    const float4 x = make_float4(x0.x * exp2_f(z.x - y.x), x0.y * exp2_f(z.y - y.y), x0.z * exp2_f(z.z - y.z), x0.w * exp2_f(z.w - y.w));
    uint32_t lo[3], hi[3];
    split3(x.x, x.y, lo);
    split3(x.z, x.w, hi);
#pragma unroll
    for (int p = 0; p < 3; ++p) *reinterpret_cast<uint2*>(kw + ((size_t)p * CQ + t) * K::LK + i) = make_uint2(lo[p], hi[p]);
  }
  __syncthreads();
  const int qr = lane >> 2, qt = lane & 3, mi = lane >> 3, r8 = lane & 7;
  const int m0 = (warp % K::MT) * 16, n0 = (warp / K::MT) * K::NW * 8;
  float acc[K::NW][4];
#pragma unroll
  for (int n = 0; n < K::NW; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
  const bf16* av = vs + ((mi >> 1) * 8 + r8) * K::LV + m0 + (mi & 1) * 8;
  const bf16* bk = kw + ((mi & 1) * 8 + r8) * K::LK + n0 + (mi >> 1) * 8;
#pragma unroll
  for (int kk = 0; kk < CQ / 16; ++kk) {
    uint32_t a[4];
    ldmatrix_x4_trans(a, av + kk * 16 * K::LV);
#pragma unroll
    for (int p = 0; p < 3; ++p)
#pragma unroll
      for (int np = 0; np < K::NW / 2; ++np) {
        uint32_t w[4];
        ldmatrix_x4_trans(w, bk + ((size_t)p * CQ + kk * 16) * K::LK + np * 16);
        mma_bf16(acc[2 * np], a, w[0], w[1]);
        mma_bf16(acc[2 * np + 1], a, w[2], w[3]);
      }
  }
  float* ug = u + (((size_t)c * H + h) * dv + col0) * dk;
#pragma unroll
  for (int n = 0; n < K::NW; ++n)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int d = m0 + qr + 8 * j, i = n0 + 8 * n + 2 * qt;
      if (d < ncols && i < dk) *reinterpret_cast<float2*>(ug + (size_t)d * dk + i) = make_float2(acc[n][2 * j], acc[n][2 * j + 1]);
    }
}

// ------------------------------------------------------------------ 2. carry
// A thread owns four state entries of a request and head.  Eight chunks' U and decays are asked for at once.
__global__ void __launch_bounds__(NTH)
gla_carry_kernel(const Request* __restrict__ requests, float* __restrict__ u, const float* __restrict__ decay, float* __restrict__ state,
                 int H, int dk, int dv) {
  const Request rq = requests[blockIdx.x / H];
  const int h = blockIdx.x % H;
  const int e = (blockIdx.y * NTH + threadIdx.x) * 4;
  if (e >= dv * dk) return;
  const int i = e % dk;
  const size_t step = (size_t)H * dv * dk, dstep = (size_t)H * dk;
  float4* sp = reinterpret_cast<float4*>(state + ((size_t)rq.slot * H + h) * dv * dk + e);
  float* up = u + ((size_t)rq.chunk0 * H + h) * dv * dk + e;
  const float* dp = decay + ((size_t)rq.chunk0 * H + h) * dk + i;
  float4 s = *sp;
  constexpr int B = 8;
  for (int c0 = 0; c0 < rq.chunks; c0 += B) {
    float4 x[B], d[B];
#pragma unroll
    for (int j = 0; j < B; ++j)
      if (c0 + j < rq.chunks) {
        x[j] = *reinterpret_cast<const float4*>(up + (size_t)(c0 + j) * step);
        d[j] = *reinterpret_cast<const float4*>(dp + (size_t)(c0 + j) * dstep);
      }
#pragma unroll
    for (int j = 0; j < B; ++j)
      if (c0 + j < rq.chunks) {
        *reinterpret_cast<float4*>(up + (size_t)(c0 + j) * step) = s;
        s = make_float4(fmaf(d[j].x, s.x, x[j].x), fmaf(d[j].y, s.y, x[j].y), fmaf(d[j].z, s.z, x[j].z), fmaf(d[j].w, s.w, x[j].w));
      }
  }
  *sp = s;
}

// ------------------------------------------------------------------ 3. outputs
// o [tokens, dv] of a chunk and head.  The scores first, by every thread; then a warp owns DVB / 8 value columns of all 64
// tokens: its share of the start state and of v it reads straight from memory, asked for before the scores are made.
template <int NT, int DVB>
struct OutShape {
  static constexpr int LB = NT + 4, LK = NT + 8, LA = CQ + 8;
  static constexpr int NW = DVB / 64;                      // column tiles of 8 a warp
  static constexpr size_t ROWS = (size_t)CQ * LB * 4;      // 64 rows of float32
  static constexpr size_t SMEM = 3 * ROWS + (size_t)(CQ - SB + SB) * LB * 4 + (size_t)(CQ / SB) * NT * 4 + (size_t)3 * CQ * LA * 2;
  static_assert((size_t)3 * CQ * LK * 2 <= ROWS + (size_t)(CQ - SB) * LB * 4, "the decayed queries lie where the keys lay");
};

template <int NT, int DVB>
__global__ void __launch_bounds__(NTH, NT <= 64 ? 2 : 1)
gla_out_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v, long long ld,
               const float* __restrict__ la, const Chunk* __restrict__ chunks, const float* __restrict__ start, float* __restrict__ out,
               int H, int dk, int dv, float q_scale) {
  using K = OutShape<NT, DVB>;
  constexpr int LB = K::LB, LK = K::LK, LA = K::LA, NW = K::NW, C4 = NT / 4;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  float* qs = reinterpret_cast<float*>(smem_raw);          // [CQ][LB] q times its scale
  float* b = qs + CQ * LB;                                 // [CQ][LB]
  float* ks = b + CQ * LB;                                 // [CQ][LB]
  float* kp = ks + CQ * LB;                                // [CQ - SB][LB] keys decayed up to a boundary
  float* qp = kp + (CQ - SB) * LB;                         // [SB][LB] queries decayed from it on
  float* tot = qp + SB * LB;                               // [CQ / SB][NT]
  bf16* as = reinterpret_cast<bf16*>(tot + (CQ / SB) * NT);     // [3][CQ][LA] the scores in three pieces
  bf16* qw = reinterpret_cast<bf16*>(ks);                  // [3][CQ][LK] the queries decayed from the chunk's start, over ks and kp
  const int c = blockIdx.x / H, h = blockIdx.x % H;
  const Chunk ch = chunks[c];
  const int col0 = blockIdx.y * DVB, ncols = min(DVB, dv - col0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qr = lane >> 2, qt = lane & 3, mi = lane >> 3, r8 = lane & 7;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);

  // the warp's columns of the start state and of v, as the products' second operands
  float2 S[NT / 16][NW][2];
  uint32_t V[CQ / 16][NW][2];
#pragma unroll
  for (int n = 0; n < NW; ++n) {
    const int d = (warp * NW + n) * 8 + qr;
    const bool in = d < ncols;
    const float* sp = start + (((size_t)c * H + h) * dv + col0 + d) * dk + 2 * qt;
#pragma unroll
    for (int kk = 0; kk < NT / 16; ++kk)
#pragma unroll
      for (int j = 0; j < 2; ++j)
        S[kk][n][j] = in && kk * 16 + 8 * j < dk ? *reinterpret_cast<const float2*>(sp + kk * 16 + 8 * j) : make_float2(0.f, 0.f);
    const float* vp = v + (size_t)ch.row0 * ld + (size_t)h * dv + col0 + d;
#pragma unroll
    for (int kk = 0; kk < CQ / 16; ++kk)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int t = kk * 16 + 8 * j + 2 * qt;
        V[kk][n][j] = pack(in && t < ch.count ? vp[(size_t)t * ld] : 0.f, in && t + 1 < ch.count ? vp[(size_t)(t + 1) * ld] : 0.f);
      }
  }

#pragma unroll 4
  for (int e = tid; e < CQ * C4; e += NTH) {
    const int t = e / C4, i = (e % C4) * 4;
    const bool in = t < ch.count && i < dk;
    const size_t at = (size_t)(ch.row0 + t) * ld + (size_t)h * dk + i;
    float4 x = in ? *reinterpret_cast<const float4*>(q + at) : zero;
    *reinterpret_cast<float4*>(qs + t * LB + i) = make_float4(x.x * q_scale, x.y * q_scale, x.z * q_scale, x.w * q_scale);
    *reinterpret_cast<float4*>(ks + t * LB + i) = in ? *reinterpret_cast<const float4*>(k + at) : zero;
    *reinterpret_cast<float4*>(b + t * LB + i) = in ? *reinterpret_cast<const float4*>(la + ((size_t)(ch.row0 + t) * H + h) * dk + i) : zero;
  }
  __syncthreads();
  cumulate<NT, LB>(b, tot);

  const int st = tid / SB, ss = tid % SB;                  // a thread's token and key within a block of the scores
  auto put = [&](int t, int s, float a) {
#pragma unroll
    for (int p = 0; p < 3; ++p) {
      const bf16 x = __float2bfloat16_rn(a);
      as[((size_t)p * CQ + t) * LA + s] = x;
      a -= __bfloat162float(x);
    }
  };
  // blocks on the diagonal
#pragma unroll 1
  for (int blk = 0; blk < CQ / SB; ++blk) {
    const int t = blk * SB + st, s = blk * SB + ss;
    float a = 0.f;
    if (ss <= st) {
      const float4 *q4 = reinterpret_cast<const float4*>(qs + t * LB), *k4 = reinterpret_cast<const float4*>(ks + s * LB);
      const float4 *bt = reinterpret_cast<const float4*>(b + t * LB), *bs = reinterpret_cast<const float4*>(b + s * LB);
#pragma unroll 4
      for (int i = 0; i < C4; ++i) {
        const float4 x = q4[i], y = k4[i], z = bt[i], w = bs[i];
        a = fmaf(x.x * y.x, exp2_f(z.x - w.x), a);
        a = fmaf(x.y * y.y, exp2_f(z.y - w.y), a);
        a = fmaf(x.z * y.z, exp2_f(z.z - w.z), a);
        a = fmaf(x.w * y.w, exp2_f(z.w - w.w), a);
      }
    }
    put(t, s, a);
  }
  // blocks below it, a row of blocks at a time
#pragma unroll
  for (int r = 1; r < CQ / SB; ++r) {
    const float* ref = b + (r * SB - 1) * LB;
    for (int e = tid; e < (r + 1) * SB * C4; e += NTH) {
      const int t = e / C4, i = (e % C4) * 4;
      const float4 z = *reinterpret_cast<const float4*>(ref + i), y = *reinterpret_cast<const float4*>(b + t * LB + i);
      const bool key = t < r * SB;
      const float4 x = *reinterpret_cast<const float4*>((key ? ks : qs) + t * LB + i);
      const float sg = key ? 1.f : -1.f;
      *reinterpret_cast<float4*>(key ? kp + t * LB + i : qp + (t - r * SB) * LB + i) =
          make_float4(x.x * exp2_f(sg * (z.x - y.x)), x.y * exp2_f(sg * (z.y - y.y)), x.z * exp2_f(sg * (z.z - y.z)), x.w * exp2_f(sg * (z.w - y.w)));
    }
    __syncthreads();
    float a[CQ / SB - 1] = {0.f, 0.f, 0.f};
    const float4* q4 = reinterpret_cast<const float4*>(qp + st * LB);
#pragma unroll 4
    for (int i = 0; i < C4; ++i) {
      const float4 x = q4[i];
#pragma unroll
      for (int j = 0; j < r; ++j) {
        const float4 y = *reinterpret_cast<const float4*>(kp + (j * SB + ss) * LB + 4 * i);
        a[j] = fmaf(x.w, y.w, fmaf(x.z, y.z, fmaf(x.y, y.y, fmaf(x.x, y.x, a[j]))));
      }
    }
#pragma unroll
    for (int j = 0; j < r; ++j) put(r * SB + st, j * SB + ss, a[j]);
    __syncthreads();
  }
  // the queries decayed from the chunk's start on
  for (int e = tid; e < CQ * C4; e += NTH) {
    const int t = e / C4, i = (e % C4) * 4;
    const float4 x = *reinterpret_cast<const float4*>(qs + t * LB + i), y = *reinterpret_cast<const float4*>(b + t * LB + i);
    uint32_t lo[3], hi[3];
    split3(x.x * exp2_f(y.x), x.y * exp2_f(y.y), lo);
    split3(x.z * exp2_f(y.z), x.w * exp2_f(y.w), hi);
#pragma unroll
    for (int p = 0; p < 3; ++p) *reinterpret_cast<uint2*>(qw + ((size_t)p * CQ + t) * LK + i) = make_uint2(lo[p], hi[p]);
  }
  __syncthreads();

  float acc[CQ / 16][NW][4];
#pragma unroll
  for (int m = 0; m < CQ / 16; ++m)
#pragma unroll
    for (int n = 0; n < NW; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][n][e] = 0.f;
  const int arow = r8 + (mi & 1) * 8, acol = (mi >> 1) * 8;
#pragma unroll
  for (int kk = 0; kk < NT / 16; ++kk) {
    uint32_t w[NW][2][3];
#pragma unroll
    for (int n = 0; n < NW; ++n)
#pragma unroll
      for (int j = 0; j < 2; ++j) split3(S[kk][n][j].x, S[kk][n][j].y, w[n][j]);
#pragma unroll
    for (int m = 0; m < CQ / 16; ++m)
#pragma unroll
      for (int p = 0; p < 3; ++p) {
        uint32_t a[4];
        ldmatrix_x4(a, qw + ((size_t)p * CQ + m * 16 + arow) * LK + kk * 16 + acol);
#pragma unroll
        for (int n = 0; n < NW; ++n)
#pragma unroll
          for (int pb = 0; pb < 3 - p; ++pb) mma_bf16(acc[m][n], a, w[n][0][pb], w[n][1][pb]);
      }
  }
#pragma unroll
  for (int kk = 0; kk < CQ / 16; ++kk)
#pragma unroll
    for (int m = kk; m < CQ / 16; ++m)
#pragma unroll
      for (int p = 0; p < 3; ++p) {
        uint32_t a[4];
        ldmatrix_x4(a, as + ((size_t)p * CQ + m * 16 + arow) * LA + kk * 16 + acol);
#pragma unroll
        for (int n = 0; n < NW; ++n) mma_bf16(acc[m][n], a, V[kk][n][0], V[kk][n][1]);
      }
  float* op = out + (size_t)ch.row0 * H * dv + (size_t)h * dv + col0;
#pragma unroll
  for (int m = 0; m < CQ / 16; ++m)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int t = m * 16 + qr + 8 * j;
      if (t >= ch.count) continue;
#pragma unroll
      for (int n = 0; n < NW; ++n) {
        const int d = (warp * NW + n) * 8 + 2 * qt;
        if (d < ncols) *reinterpret_cast<float2*>(op + (size_t)t * H * dv + d) = make_float2(acc[m][n][2 * j], acc[m][n][2 * j + 1]);
      }
    }
}

namespace {

template <int NT, int DVB>
int run_chunks(const float* q, const float* k, const float* v, long long ld, const float* la, const Chunk* chunks, int n_chunks,
               const Request* requests, int n_requests, float* u, float* decay, float* state, float* out, int H, int dk, int dv,
               float q_scale, cudaStream_t s) {
  const dim3 grid((unsigned)(n_chunks * H), (unsigned)((dv + DVB - 1) / DVB));
  static HkSmemCache c1, c3;
  if (int e = hk_allow_smem(gla_states_kernel<NT, DVB>, StatesShape<NT, DVB>::SMEM, c1)) return e;
  if (int e = hk_allow_smem(gla_out_kernel<NT, DVB>, OutShape<NT, DVB>::SMEM, c3)) return e;
  if (int e = hk_launch(gla_states_kernel<NT, DVB>, grid, dim3(NTH), StatesShape<NT, DVB>::SMEM, s, k, v, ld, la, chunks, u, decay, H, dk, dv))
    return e;
  if (int e = hk_launch(gla_carry_kernel, dim3((unsigned)(n_requests * H), (unsigned)((dv * dk / 4 + NTH - 1) / NTH)), dim3(NTH), 0, s, requests, u,
                        decay, state, H, dk, dv))
    return e;
  return hk_launch(gla_out_kernel<NT, DVB>, grid, dim3(NTH), OutShape<NT, DVB>::SMEM, s, q, k, v, ld, la, chunks, u, out, H, dk, dv, q_scale);
}

}  // namespace

// q, k [n, H dk] and v [n, H dv]: column slices of one float32 matrix (row stride ld); la float32 [n, H dk]; chunks int32
// [n_chunks, 2] = (first row, rows <= 64), a request's chunks one after the other and all but its last of 64 rows; requests
// int32 [n_requests, 3] = (state slot, first chunk, chunks); u float32 [n_chunks, H, dv, dk] and decay float32 [n_chunks, H, dk]
// scratch; state float32 [slots, H, dv, dk]; out float32 [n, H dv].  Refuses (HK_ERR_UNSUPPORTED) what the 16-byte copies
// cannot take (dk or dv no multiple of 8, rows or pointers off a 16-byte boundary) and keys above 128.
HK_API int hk_gla_chunks(const float* q, const float* k, const float* v, long long ld, const float* la, const int* chunks, int n_chunks,
                         const int* requests, int n_requests, float* u, float* decay, float* state, float* out, int H, int dk, int dv,
                         float q_scale, void* stream) {
  if (n_chunks <= 0 || n_requests <= 0) return 0;
  if (H < 1 || dk < 8 || dk > 128 || (dk & 7) || dv < 8 || (dv & 7) || (ld & 3)) return HK_ERR_UNSUPPORTED;
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)la | (uintptr_t)u | (uintptr_t)decay | (uintptr_t)state | (uintptr_t)out) & 15)
    return HK_ERR_UNSUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
#define CHUNKS(NT, DVB)                                                                                                              \
  run_chunks<NT, DVB>(q, k, v, ld, la, (const Chunk*)chunks, n_chunks, (const Request*)requests, n_requests, u, decay, state, out, H, dk, dv, \
                      q_scale, s)
  // 128 columns a block share the scores; 64 where there are no more
  if (dk <= 32) return dv > 64 ? CHUNKS(32, 128) : CHUNKS(32, 64);
  if (dk <= 64) return dv > 64 ? CHUNKS(64, 128) : CHUNKS(64, 64);
  return dv > 64 ? CHUNKS(128, 128) : CHUNKS(128, 64);
#undef CHUNKS
}
