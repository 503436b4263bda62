// The scans of gated linear attention (a decay per key channel) and of the gated delta rule with one decay per head, for long
// portions in bfloat16 mode, 16 tokens at a time on tensor cores (mma.sync m16n8k16). With L_t the sum of the logarithms of
// the chunk's decays up to token t (per key channel c or per head) and S the state before the chunk,
//
//   o_t = S^T (q_t e^{L_t}) + sum_{s <= t} P_ts u_s,      P_ts = sum_c q_tc k_sc e^{L_tc - L_sc}
//   S  <- e^{L_16} S + sum_s (k_s e^{L_16 - L_s}) u_s^T
//
// where u_s = v_s for linear attention. The delta rule's u_s = beta_s (v_s - (what the state returns under k_s before the write))
// solves (I + M) U = diag(beta) (V - (K e^L) S) with M_ts = beta_t e^{L_t - L_s} (k_t . k_s) for s < t, so with T = (I + M)^-1
//
//   U = V' - W S,      V' = T diag(beta) V,      W = T diag(beta) (K e^L),
//
// which is the token-by-token recurrence (gla.cu, seq_mix.cu) in another order: T is lower triangular with ones on the diagonal
// and is found by substitution in 32-bit. Every exponent is a sum of logarithms of decays between two tokens of the chunk, s
// <= t, so at most zero: no quotient of decays is formed and nothing overflows however fast a channel forgets.
//
// Two kernels. The first has a block per (chunk, head), all independent: decays, unit vectors, P, T, W and V' in 32-bit, left in
// a record of scratch memory as operands of matrix products, each 32-bit number as the sum of two bfloat16 numbers (its
// rounding and the rounding of what is left; the products of two rests are dropped: a relative error of 2^-17 per term). The
// second walks a portion's chunks in order: a block owns 32 value columns of a head of a portion, and each of its four warps
// keeps 16 of them x half of the key channels of S^T in its accumulators from the portion's first chunk to its last. As the
// first operand of the products with Q and W, and with U^T as the first operand of the products with P and K, the accumulators'
// own layout is that of the operand, so the state never leaves the registers. What the two halves of the key channels add up
// to (o, and for the delta rule W S) passes through shared memory. A chunk's record, and the block's columns of V, travel to
// shared memory in one bulk copy each, two chunks ahead; the first kernel writes them in the layout they are used in.
#include "attn_mma.cuh"
#include "tma.cuh"
#include <math.h>

namespace {
using namespace fzattn;
constexpr int C = 16;                       // tokens per chunk
constexpr int COOK_THREADS = 256;
constexpr int SLICE = 32;                   // value columns per block of the second kernel
constexpr int STAGES = 6;                  // chunks in shared memory at a time
constexpr float LOG2E = 1.4426950408889634f;

// 2^x for x <= 0 (results below the normal range are zero)
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float softplus32(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// Two 32-bit values as bfloat16 pairs: their roundings, and the roundings of what is left.
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  hi = *(const uint32_t*)&h;
  lo = pack_bf16(a - f.x, b - f.y);
}

// The record of a (chunk, head), in bytes. Main part: MATS matrices [16][DKP] of bf16 (Q, K and for the delta rule W; rounding,
// then rest), P [16][16] (rounding, rest), the chunk's decays (DKP floats). Then V in slices of 32 columns: rounding and rest
// [16][32] bf16 (linear attention) or V' [16][32] float (delta rule). Every row is 16 bytes longer than its values (an odd
// number of 16-byte units: the rows that are read together from shared memory fall into different banks).
template <int DKP, bool DELTA> struct Record {
  static constexpr int MATS = DELTA ? 6 : 4, ROW = DKP * 2 + 16, MAT = C * ROW, P_ROW = C * 2 + 16, P_MAT = C * P_ROW;
  static constexpr int P = MATS * MAT, DECAY = P + 2 * P_MAT, MAIN = DECAY + DKP * 4;
  static constexpr int V_ROW = SLICE * (DELTA ? 4 : 2) + 16, V_MAT = C * V_ROW, V = (DELTA ? 1 : 2) * V_MAT;
  static constexpr int STAGE = MAIN + V;
};
__host__ __device__ inline int slices_of(int dv) { return (dv + SLICE - 1) / SLICE; }
template <int DKP, bool DELTA> __host__ __device__ inline long long record_bytes(int dv) {
  return Record<DKP, DELTA>::MAIN + (long long)slices_of(dv) * Record<DKP, DELTA>::V;
}
// The records of a portion that begins at row r stand from place ceil(r / 8) on. A portion of n >= 16 rows has ceil(n / 16) of
// them, and ceil((r + n) / 8) >= ceil(r / 8) + ceil((n - 7) / 8) >= ceil(r / 8) + ceil(n / 16): no two portions of 16 rows and
// more share a place, and a step of N rows needs ceil(N / 8) places, whatever portions it holds.
__device__ __forceinline__ long long record_place(int row0, int chunk) { return (row0 + 7) / 8 + chunk; }

// A [16][DKP] matrix as rounding (matrix `m` of the record) and rest (the one after it); value2(t, c): elements c and c + 1.
template <int DKP, bool DELTA, typename Fn>
__device__ __forceinline__ void leave_matrix(unsigned char* rec, int m, Fn value2) {
  using R = Record<DKP, DELTA>;
  const int c = 2 * (threadIdx.x % (DKP / 2));
#pragma unroll
  for (int t = threadIdx.x / (DKP / 2); t < C; t += 2 * COOK_THREADS / DKP) {
    const float2 v = value2(t, c);
    uint32_t h, l;
    split2(v.x, v.y, h, l);
    *(uint32_t*)(rec + m * R::MAT + t * R::ROW + 2 * c) = h;
    *(uint32_t*)(rec + (m + 1) * R::MAT + t * R::ROW + 2 * c) = l;
  }
}
// Row t of P, whose element `lane` is v: rounding and rest.
template <typename R>
__device__ __forceinline__ void leave_p(unsigned char* rec, int t, int lane, float v) {
  const __nv_bfloat16 hi = __float2bfloat16_rn(v);
  *(__nv_bfloat16*)(rec + R::P + t * R::P_ROW + 2 * lane) = hi;
  *(__nv_bfloat16*)(rec + R::P + R::P_MAT + t * R::P_ROW + 2 * lane) = __float2bfloat16_rn(v - __bfloat162float(hi));
}

struct CookArgs {
  const int* seg;
  int H, Hk, dk, dv, min_rows;
  unsigned char* scratch;
  // linear attention: proj rows of ld floats [q heads | k heads | v heads | ...], z rows of H dk decay inputs
  const float* proj;
  int ld;
  const float* z;
  float inv_root;
  // delta rule: qkv rows [q (Hk dk) | k (Hk dk) | v (H dv)] of bf16; decay inputs and betas, one per head
  const __nv_bfloat16* qkv;
  const float* high;
  int ldh;
  const float* beta;
  int ldb;
  const float *a_log, *dt_bias;
  float unit_eps;
  float q_scale;
};

// grid (portions, chunks of the longest portion, heads)
template <int DKP>
__global__ void __launch_bounds__(COOK_THREADS)
gla_cook_kernel(const CookArgs a) {
  using R = Record<DKP, false>;
  fz_grid_launch_dependents();
  const int s = blockIdx.x, c0 = blockIdx.y * C, h = blockIdx.z;
  const int row0 = a.seg[4 * s], cnt = a.seg[4 * s + 1], slot = a.seg[4 * s + 3];
  fz_grid_wait();
  if (cnt < a.min_rows || c0 >= cnt || slot < 0) return;
  constexpr int LD = DKP + 4;
  __shared__ __align__(16) float q[C * LD], k[C * LD], L[C * LD];      // L: logarithms (base 2) of the decays, then their running sums
  const int dk = a.dk, valid = min(C, cnt - c0), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  unsigned char* rec = a.scratch + (record_place(row0, blockIdx.y) * a.H + h) * record_bytes<DKP, false>(a.dv);
  const size_t n0 = (size_t)(row0 + c0);
  {
    const int c = tid % DKP;
#pragma unroll
    for (int t = tid / DKP; t < C; t += COOK_THREADS / DKP) {
      float qv = 0.f, kv = 0.f, lv = 0.f;
      if (c < dk && t < valid) {
        const float* in = a.proj + (n0 + t) * a.ld;
        qv = __fmul_rn(in[(size_t)h * dk + c], a.q_scale);
        kv = in[(size_t)(a.H + h) * dk + c];
        lv = -a.inv_root * softplus32(-a.z[(n0 + t) * a.H * dk + (size_t)h * dk + c]) * LOG2E;
      }
      q[t * LD + c] = qv;
      k[t * LD + c] = kv;
      L[t * LD + c] = lv;
    }
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {         // V needs nothing of the above
    const int t = warp + 8 * half;
    const float* in = a.proj + (n0 + t) * a.ld + (size_t)2 * a.H * dk + (size_t)h * a.dv;
    for (int c = 2 * lane; c < slices_of(a.dv) * SLICE; c += 64) {
      uint32_t hi, lo;
      split2(t < valid && c < a.dv ? in[c] : 0.f, t < valid && c + 1 < a.dv ? in[c + 1] : 0.f, hi, lo);
      unsigned char* v = rec + R::MAIN + (c / SLICE) * R::V + t * R::V_ROW + (c % SLICE) * 2;
      *(uint32_t*)v = hi;
      *(uint32_t*)(v + R::V_MAT) = lo;
    }
  }
  __syncthreads();
  if (tid < DKP) {
    float run = 0.f;
#pragma unroll
    for (int t = 0; t < C; ++t) { run += L[t * LD + tid]; L[t * LD + tid] = run; }
    ((float*)(rec + R::DECAY))[tid] = ex2(run);
  }
  __syncthreads();
  auto at = [&](const float* m, int t, int c) { return *(const float2*)(m + t * LD + c); };
  leave_matrix<DKP, false>(rec, 0, [&](int t, int c) {
    const float2 x = at(q, t, c), l = at(L, t, c);
    return make_float2(x.x * ex2(l.x), x.y * ex2(l.y));
  });
  leave_matrix<DKP, false>(rec, 2, [&](int t, int c) {
    const float2 x = at(k, t, c), l = at(L, t, c), e = at(L, C - 1, c);
    return make_float2(x.x * ex2(e.x - l.x), x.y * ex2(e.y - l.y));
  });
  const int c = 4 * lane;                        // this lane's four key channels
  const bool in = c < DKP;
  const float4 none = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int half = 0; half < 2; ++half) {         // a warp takes token `warp` and token 15 - `warp`: 17 pairs
    const int t = half == 0 ? warp : C - 1 - warp;
    const float4 qt = in ? *(const float4*)(q + t * LD + c) : none, Lt = in ? *(const float4*)(L + t * LD + c) : none;
    float mine = 0.f;                            // lane s keeps P_ts
    for (int x = 0; x <= t; ++x) {
      const float4 kx = in ? *(const float4*)(k + x * LD + c) : none, Lx = in ? *(const float4*)(L + x * LD + c) : none;
      float acc = qt.x * kx.x * ex2(Lt.x - Lx.x);
      acc = fmaf(qt.y * kx.y, ex2(Lt.y - Lx.y), acc);
      acc = fmaf(qt.z * kx.z, ex2(Lt.z - Lx.z), acc);
      acc = fmaf(qt.w * kx.w, ex2(Lt.w - Lx.w), acc);
      acc = warp_sum(acc);
      if (lane == x) mine = acc;
    }
    if (lane < C) leave_p<R>(rec, t, lane, mine);
  }
}

template <int DKP>
__global__ void __launch_bounds__(COOK_THREADS)
delta_cook_kernel(const CookArgs a) {
  using R = Record<DKP, true>;
  fz_grid_launch_dependents();
  const int s = blockIdx.x, c0 = blockIdx.y * C, h = blockIdx.z;
  const int row0 = a.seg[4 * s], cnt = a.seg[4 * s + 1], slot = a.seg[4 * s + 3];
  const float rate2 = expf(a.a_log[h]) * LOG2E, bias = a.dt_bias[h];
  fz_grid_wait();
  if (cnt < a.min_rows || c0 >= cnt || slot < 0) return;
  constexpr int LD = DKP + 4, TP = 17;
  __shared__ __align__(16) float q[C * LD], k[C * LD];
  __shared__ float M[C * TP], T1[C * TP], T2[C * TP], L[C], b[C];      // M: beta_t e^{L_t - L_s} k_t . k_s below the diagonal; T1: T diag(beta), T2: T diag(beta e^L)
  extern __shared__ __align__(16) float v[];     // [16][columns of V, to a multiple of 32]
  const int dk = a.dk, valid = min(C, cnt - c0), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int dvp = slices_of(a.dv) * SLICE;
  unsigned char* rec = a.scratch + (record_place(row0, blockIdx.y) * a.H + h) * record_bytes<DKP, true>(a.dv);
  const size_t n0 = (size_t)(row0 + c0);
  const int kh = h / (a.H / a.Hk), W = 2 * a.Hk * dk + a.H * a.dv;
  constexpr int PER = (DKP + 31) / 32;           // key channels per lane
#pragma unroll
  for (int half = 0; half < 2; ++half) {         // a warp brings two tokens in: unit vectors, values
    const int t = warp + 8 * half;
    const __nv_bfloat16* in = a.qkv + (n0 + t) * W;
    float qv[PER], kv[PER], sq = 0.f, sk = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int c = lane + 32 * i;
      const bool ok = c < dk && t < valid;
      qv[i] = ok ? __bfloat162float(in[(size_t)kh * dk + c]) : 0.f;
      kv[i] = ok ? __bfloat162float(in[(size_t)(a.Hk + kh) * dk + c]) : 0.f;
      sq = fmaf(qv[i], qv[i], sq);
      sk = fmaf(kv[i], kv[i], sk);
    }
    const float nq = sqrtf(warp_sum(sq) + a.unit_eps), nk = sqrtf(warp_sum(sk) + a.unit_eps);
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int c = lane + 32 * i;
      if (c < DKP) {
        q[t * LD + c] = __fmul_rn(__fdiv_rn(qv[i], nq), a.q_scale);
        k[t * LD + c] = __fdiv_rn(kv[i], nk);
      }
    }
    const __nv_bfloat16* vin = in + (size_t)2 * a.Hk * dk + (size_t)h * a.dv;
    for (int c = lane; c < dvp; c += 32) v[t * dvp + c] = t < valid && c < a.dv ? __bfloat162float(vin[c]) : 0.f;
  }
  if (warp == 0) {
    float l = 0.f, be = 0.f;
    if (lane < valid) {
      l = -rate2 * softplus32(a.high[(n0 + lane) * a.ldh + h] + bias);
      be = 1.0f / (1.0f + expf(-a.beta[(n0 + lane) * a.ldb + h]));
    }
#pragma unroll
    for (int o = 1; o < C; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, l, o);
      if (lane >= o) l += y;
    }
    if (lane < C) { L[lane] = l; b[lane] = be; }
  }
  __syncthreads();
  const int c = 4 * lane;                        // this lane's four key channels
  const bool in = c < DKP;
  const float4 none = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = half == 0 ? warp : C - 1 - warp;
    const float4 qt = in ? *(const float4*)(q + t * LD + c) : none, kt = in ? *(const float4*)(k + t * LD + c) : none;
    float qk = 0.f, kk = 0.f;                    // lane s keeps the products with k_s
    for (int x = 0; x <= t; ++x) {
      const float4 kx = in ? *(const float4*)(k + x * LD + c) : none;
      const float p = warp_sum(fmaf(qt.x, kx.x, fmaf(qt.y, kx.y, fmaf(qt.z, kx.z, qt.w * kx.w))));
      const float m = warp_sum(fmaf(kt.x, kx.x, fmaf(kt.y, kx.y, fmaf(kt.z, kx.z, kt.w * kx.w))));
      if (lane == x) { qk = p; kk = m; }
    }
    if (lane < C) {
      const float f = lane <= t ? ex2(L[t] - L[lane]) : 0.f;
      leave_p<R>(rec, t, lane, qk * f);
      M[t * TP + lane] = lane < t ? b[t] * f * kk : 0.f;
    }
  }
  __syncthreads();
  if (tid < C) {                                 // column j of T by substitution: T_tj = [t = j] - sum_{s < t} M_ts T_sj
    const int j = tid;
    float x[C];
#pragma unroll
    for (int t = 0; t < C; ++t) {
      float acc = t == j ? 1.f : 0.f;
#pragma unroll
      for (int y = 0; y < t; ++y) acc = fmaf(-M[t * TP + y], x[y], acc);
      x[t] = acc;
    }
    const float b1 = b[j], b2 = b1 * ex2(L[j]);
#pragma unroll
    for (int t = 0; t < C; ++t) { T1[t * TP + j] = x[t] * b1; T2[t * TP + j] = x[t] * b2; }
  }
  const float last = L[C - 1];
  auto at = [&](const float* m, int t, int c) { return *(const float2*)(m + t * LD + c); };
  leave_matrix<DKP, true>(rec, 0, [&](int t, int c) {
    const float2 x = at(q, t, c);
    const float f = ex2(L[t]);
    return make_float2(x.x * f, x.y * f);
  });
  leave_matrix<DKP, true>(rec, 2, [&](int t, int c) {
    const float2 x = at(k, t, c);
    const float f = ex2(last - L[t]);
    return make_float2(x.x * f, x.y * f);
  });
  if (tid < DKP) ((float*)(rec + R::DECAY))[tid] = ex2(last);
  __syncthreads();
  leave_matrix<DKP, true>(rec, 4, [&](int t, int c) {
    float2 acc = make_float2(0.f, 0.f);
    for (int y = 0; y <= t; ++y) {
      const float2 x = at(k, y, c);
      const float f = T2[t * TP + y];
      acc.x = fmaf(f, x.x, acc.x);
      acc.y = fmaf(f, x.y, acc.y);
    }
    return acc;
  });
#pragma unroll
  for (int half = 0; half < 2; ++half) {         // a warp takes token `warp` and token 15 - `warp`: 17 terms in all
    const int t = half == 0 ? warp : C - 1 - warp;
    for (int c = lane; c < dvp; c += 32) {
      float acc = 0.f;
      for (int y = 0; y <= t; ++y) acc = fmaf(T1[t * TP + y], v[y * dvp + c], acc);
      *(float*)(rec + R::MAIN + (c / SLICE) * R::V + t * R::V_ROW + (c % SLICE) * 4) = acc;
    }
  }
}

__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void pair_barrier(int id) { asm volatile("bar.sync %0, 64;" ::"r"(id) : "memory"); }

// ---- the second kernel: grid (portions, heads, slices of 32 value columns), 64 KS threads: warp w owns columns 16 (w % 2) ..
// + 15 of the slice and part w / 2 of the KS parts of the key channels.
template <int DKP, bool DELTA, int KS>
__global__ void __launch_bounds__(64 * KS)
scan_chunk_kernel(const unsigned char* __restrict__ scratch, int H, int dv, float* __restrict__ state, const int* __restrict__ seg,
                  int min_rows, float* __restrict__ out, int* err) {
  using R = Record<DKP, DELTA>;
  fz_grid_launch_dependents();
  const int s = blockIdx.x, h = blockIdx.y, slice = blockIdx.z;
  const int row0 = seg[4 * s], cnt = seg[4 * s + 1], slot = seg[4 * s + 3];
  fz_grid_wait();
  if (cnt < min_rows || cnt <= 0 || slot < 0) return;
  extern __shared__ __align__(128) unsigned char smem[];
  __shared__ uint64_t full[STAGES];
  __shared__ float xo[KS > 1 ? 2 : 1][2][8][32];                 // results of the second half of the key channels, by chunk parity
  __shared__ float xd[DELTA && KS > 1 ? 2 * KS : 1][8][32];      // a warp's part of W S
  const uint32_t s0 = smem_u32(smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, cg = warp & 1, kh = warp >> 1;
  const int g = lane >> 2, q2 = 2 * (lane & 3);            // an accumulator's row (and row + 8) and first column
  const int nc = (cnt + C - 1) / C;
  const long long bytes = record_bytes<DKP, DELTA>(dv), step = (long long)H * bytes;
  const unsigned char* base = scratch + (record_place(row0, 0) * H + h) * bytes;

  if (tid == 0) {
    for (int i = 0; i < STAGES; ++i) fztma::mbar_init(&full[i], 1);
    fztma::mbar_init_fence();
  }
  auto issue = [&](int c) {                                // one thread
    const unsigned char* r = base + c * step;
    const uint32_t st = s0 + (c % STAGES) * R::STAGE;
    uint64_t* bar = &full[c % STAGES];
    fztma::mbar_expect_tx(bar, R::STAGE);
    bulk_load(st, r, R::MAIN, bar);
    bulk_load(st + R::MAIN, r + R::MAIN + (long long)slice * R::V, R::V, bar);
  };
  if (tid == 0)
    for (int c = 0; c < STAGES - 1 && c < nc; ++c) issue(c);

  constexpr int KN = DKP / 16 / KS;                        // 16-channel steps of this warp
  const int k0 = kh * KN;
  float S[2 * KN][4];                                      // S^T: rows are value columns, columns are key channels
  const int ca = slice * SLICE + 16 * cg + g, cb = ca + 8; // this thread's two value columns
  float* sa = state + (((size_t)slot * H + h) * dv + ca) * DKP + 16 * k0 + q2;
  float* sb = sa + (size_t)8 * DKP;
#pragma unroll
  for (int n = 0; n < 2 * KN; ++n) {
    const float2 x = ca < dv ? *(const float2*)(sa + 8 * n) : make_float2(0.f, 0.f);
    const float2 y = cb < dv ? *(const float2*)(sb + 8 * n) : make_float2(0.f, 0.f);
    S[n][0] = x.x; S[n][1] = x.y; S[n][2] = y.x; S[n][3] = y.y;
  }
  const int mi = lane >> 3, l7 = lane & 7;
  // rows of operands whose 16 rows are the product's columns (Q, W, P), and of those whose rows are summed over (K, V)
  const uint32_t off_n = ((mi >> 1) * 8 + l7), off_k = ((mi & 1) * 8 + l7);
  float O[2][4];                                           // results of the chunk in hand (columns x tokens)
  auto leave_results = [&](int c) {                        // by the warps of the first part: theirs and the second part's
    const int valid = min(C, cnt - c * C);
    float* dst = out + ((size_t)(row0 + c * C) * H + h) * dv;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = 8 * n + q2 + (e & 1), col = e < 2 ? ca : cb;
        const float y = KS > 1 ? O[n][e] + xo[c & 1][cg][4 * n + e][lane] : O[n][e];
        if (t < valid && col < dv) dst[(size_t)t * H * dv + col] = y;
      }
  };
  __syncthreads();                                         // the barriers are ready

  for (int c = 0; c < nc; ++c) {
    const bool ok = fztma::mbar_wait(&full[c % STAGES], (c / STAGES) & 1);
    if (!__syncthreads_and(ok)) {                          // (also: everyone is done with chunk c - 1)
      if (tid == 0) atomicOr(err, FZ_ERR_WAIT_TIMEOUT);
      return;
    }
    if (tid == 0 && c + STAGES - 1 < nc) issue(c + STAGES - 1);      // into the place of chunk c - 1
    if (c > 0 && kh == 0) leave_results(c - 1);
    const uint32_t st = s0 + (c % STAGES) * R::STAGE;
    const unsigned char* sp = smem + (c % STAGES) * R::STAGE;
    uint32_t hi[KN][4], lo[KN][4];                         // the state as a first operand
#pragma unroll
    for (int k = 0; k < KN; ++k) {
      split2(S[2 * k][0], S[2 * k][1], hi[k][0], lo[k][0]);
      split2(S[2 * k][2], S[2 * k][3], hi[k][1], lo[k][1]);
      split2(S[2 * k + 1][0], S[2 * k + 1][1], hi[k][2], lo[k][2]);
      split2(S[2 * k + 1][2], S[2 * k + 1][3], hi[k][3], lo[k][3]);
    }
    float acc[3][2][4];                                    // hi . hi, rest . hi, hi . rest
    auto clear = [&]() {
#pragma unroll
      for (int x = 0; x < 3; ++x)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) acc[x][n][e] = 0.f;
    };
    auto times = [&](const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t at_hi, uint32_t at_lo) {
      uint32_t bh[4], bl[4];
      ldmatrix_x4(bh, at_hi);
      ldmatrix_x4(bl, at_lo);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        mma_bf16(acc[0][n], ah, bh[2 * n], bh[2 * n + 1]);
        mma_bf16(acc[1][n], al, bh[2 * n], bh[2 * n + 1]);
        mma_bf16(acc[2][n], ah, bl[2 * n], bl[2 * n + 1]);
      }
    };
    const uint32_t a_q = st + off_n * R::ROW + (mi & 1) * 16 + 32 * k0;
    float D[2][4];
    if constexpr (DELTA) {                                 // this part of W S
      clear();
#pragma unroll
      for (int k = 0; k < KN; ++k) times(hi[k], lo[k], a_q + 4 * R::MAT + 32 * k, a_q + 5 * R::MAT + 32 * k);
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          D[n][e] = acc[0][n][e] + (acc[1][n][e] + acc[2][n][e]);
          if (KS > 1) xd[warp][4 * n + e][lane] = D[n][e];
        }
    }
    clear();
#pragma unroll
    for (int k = 0; k < KN; ++k) times(hi[k], lo[k], a_q + 32 * k, a_q + R::MAT + 32 * k);
    uint32_t uh[4], ul[4];                                 // U^T (value columns x tokens) as a first operand
    if constexpr (DELTA) {
      if (KS > 1) {
        pair_barrier(1 + cg);
#pragma unroll
        for (int i = 0; i < 8; ++i) D[i >> 2][i & 3] = xd[cg][i][lane] + xd[cg + 2][i][lane];      // (the same order in both warps)
      }
      const float* v = (const float*)(sp + R::MAIN) + 16 * cg + g;
      constexpr int VR = R::V_ROW / 4;
      float U[2][4];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) U[n][e] = v[(8 * n + q2 + (e & 1)) * VR + (e >> 1) * 8] - D[n][e];
      split2(U[0][0], U[0][1], uh[0], ul[0]);
      split2(U[0][2], U[0][3], uh[1], ul[1]);
      split2(U[1][0], U[1][1], uh[2], ul[2]);
      split2(U[1][2], U[1][3], uh[3], ul[3]);
    } else {
      const uint32_t a_v = st + R::MAIN + off_n * R::V_ROW + (16 * cg + (mi & 1) * 8) * 2;
      ldmatrix_x4_trans(uh, a_v);
      ldmatrix_x4_trans(ul, a_v + R::V_MAT);
    }
    const uint32_t a_k = st + 2 * R::MAT + off_k * R::ROW + (mi >> 1) * 16 + 32 * k0;
    const float* dec = (const float*)(sp + R::DECAY) + 16 * k0 + q2;
#pragma unroll
    for (int k = 0; k < KN; ++k) {
      uint32_t bh[4], bl[4];
      ldmatrix_x4_trans(bh, a_k + 32 * k);
      ldmatrix_x4_trans(bl, a_k + R::MAT + 32 * k);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        float* x = S[2 * k + n];
        const float2 d = *(const float2*)(dec + 16 * k + 8 * n);
        x[0] *= d.x; x[1] *= d.y; x[2] *= d.x; x[3] *= d.y;
        mma_bf16(x, uh, bh[2 * n], bh[2 * n + 1]);
        mma_bf16(x, ul, bh[2 * n], bh[2 * n + 1]);
        mma_bf16(x, uh, bl[2 * n], bl[2 * n + 1]);
      }
    }
    if (kh == KS - 1) {
      const uint32_t a_p = st + R::P + off_n * R::P_ROW + (mi & 1) * 16;
      times(uh, ul, a_p, a_p + R::P_MAT);
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        O[n][e] = acc[0][n][e] + (acc[1][n][e] + acc[2][n][e]);
        if (KS > 1 && kh == 1) xo[c & 1][cg][4 * n + e][lane] = O[n][e];
      }
  }
  __syncthreads();
  if (kh == 0) leave_results(nc - 1);
#pragma unroll
  for (int n = 0; n < 2 * KN; ++n) {
    if (ca < dv) *(float2*)(sa + 8 * n) = make_float2(S[n][0], S[n][1]);
    if (cb < dv) *(float2*)(sb + 8 * n) = make_float2(S[n][2], S[n][3]);
  }
}

int padded_keys(int dk) {                   // of the state's own layout: 8 times a power of two
  int p = 8;
  while (p < dk) p <<= 1;
  return p;
}

template <typename K>
int allow_smem(K kern, size_t smem, size_t& allowed) {
  if (smem <= allowed) return FZ_OK;
  if (smem > 227 * 1024) return FZ_TOO_LARGE;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  allowed = smem;
  return FZ_OK;
}

template <int DKP, bool DELTA>
int launch_both(const CookArgs& a, float* state, int n_seg, int max_rows, float* out, int* err, cudaStream_t stream) {
  constexpr int KS = DKP >= 32 ? 2 : 1;
  const int chunks = (max_rows + C - 1) / C;
  if (chunks > 65535) return FZ_TOO_LARGE;
  const size_t cook_smem = DELTA ? sizeof(float) * C * slices_of(a.dv) * SLICE : 0;
  constexpr size_t smem = (size_t)STAGES * Record<DKP, DELTA>::STAGE;
  static size_t allowed_c = 16 * 1024, allowed = 32 * 1024;      // (beside their static shared memory)
  auto cook = DELTA ? delta_cook_kernel<DKP> : gla_cook_kernel<DKP>;
  auto scan = scan_chunk_kernel<DKP, DELTA, KS>;
  int st = allow_smem(cook, cook_smem, allowed_c);
  if (st != FZ_OK || (st = allow_smem(scan, smem, allowed)) != FZ_OK) return st;
  fz_launch(cook, dim3(n_seg, chunks, a.H), dim3(COOK_THREADS), cook_smem, stream, a);
  FZ_LAUNCH_CHECK();
  fz_launch(scan, dim3(n_seg, a.H, slices_of(a.dv)), dim3(64 * KS), smem, stream, (const unsigned char*)a.scratch, a.H, a.dv, state, a.seg,
            a.min_rows, out, err);
  FZ_LAUNCH_CHECK();
  return FZ_OK;
}

template <bool DELTA>
int run(const CookArgs& a, float* state, int n_seg, int max_rows, float* out, int* err, cudaStream_t stream) {
  switch (padded_keys(a.dk)) {
    case 16: return launch_both<16, DELTA>(a, state, n_seg, max_rows, out, err, stream);
    case 32: return launch_both<32, DELTA>(a, state, n_seg, max_rows, out, err, stream);
    case 64: return launch_both<64, DELTA>(a, state, n_seg, max_rows, out, err, stream);
    default: return launch_both<128, DELTA>(a, state, n_seg, max_rows, out, err, stream);
  }
}
template <bool DELTA> long long bytes_of(int dkp, int dv) {
  return dkp == 16 ? record_bytes<16, DELTA>(dv) : dkp == 32 ? record_bytes<32, DELTA>(dv) : dkp == 64 ? record_bytes<64, DELTA>(dv) : record_bytes<128, DELTA>(dv);
}
}  // namespace

// Sizes taken: keys of 9 to 128, values of up to 1,024.
FZ_API int fz_scan_chunk_check(int H, int dk, int dv) {
  return (H > 0 && H <= 65535 && dk > 8 && dk <= 128 && dv > 0 && dv <= 1024) ? FZ_OK : FZ_BAD_SHAPE;
}

// Bytes of scratch for a step of N rows (see record_place).
FZ_API long long fz_scan_chunk_scratch(int N, int H, int dk, int dv, int delta) {
  const int dkp = padded_keys(dk);
  return ((long long)N / 8 + 1) * H * (delta ? bytes_of<true>(dkp, dv) : bytes_of<false>(dkp, dv));
}

// Portions of min_rows rows and more (max_rows at most); the state is (slots, H, dv, padded keys). See fz_channel_decay_scan.
FZ_API int fz_gla_chunk(const float* proj, int ld, int H, int dk, int dv, const float* z, float inv_root, float q_scale, float* state,
                        const int* seg, int n_seg, int min_rows, int max_rows, void* scratch, float* out, int* err, cudaStream_t stream) {
  if (n_seg <= 0) return FZ_OK;
  if (fz_scan_chunk_check(H, dk, dv) != FZ_OK || ld < H * (2 * dk + dv) || scratch == nullptr || ((uintptr_t)scratch & 15) || min_rows < C) return FZ_BAD_SHAPE;
  CookArgs a = {};
  a.seg = seg; a.H = a.Hk = H; a.dk = dk; a.dv = dv; a.min_rows = min_rows; a.scratch = (unsigned char*)scratch;
  a.proj = proj; a.ld = ld; a.z = z; a.inv_root = inv_root; a.q_scale = q_scale;
  return run<false>(a, state, n_seg, max_rows, out, err, stream);
}

// See fz_gated_delta_scan (one decay per head).
FZ_API int fz_delta_chunk(const void* qkv, int H, int Hk, int dk, int dv, const float* high, int ldh, const float* beta, int ldb,
                          const float* a_log, const float* dt_bias, float unit_eps, float q_scale, float* state, const int* seg,
                          int n_seg, int min_rows, int max_rows, void* scratch, float* out, int* err, cudaStream_t stream) {
  if (n_seg <= 0) return FZ_OK;
  if (fz_scan_chunk_check(H, dk, dv) != FZ_OK || Hk <= 0 || H % Hk || scratch == nullptr || ((uintptr_t)scratch & 15) || min_rows < C) return FZ_BAD_SHAPE;
  CookArgs a = {};
  a.seg = seg; a.H = H; a.Hk = Hk; a.dk = dk; a.dv = dv; a.min_rows = min_rows; a.scratch = (unsigned char*)scratch;
  a.qkv = (const __nv_bfloat16*)qkv; a.high = high; a.ldh = ldh; a.beta = beta; a.ldb = ldb; a.a_log = a_log; a.dt_bias = dt_bias;
  a.unit_eps = unit_eps; a.q_scale = q_scale;
  return run<true>(a, state, n_seg, max_rows, out, err, stream);
}

#ifdef FZ_TIMELINE
FZ_TIMELINE_READER(scan_chunk)
#endif
