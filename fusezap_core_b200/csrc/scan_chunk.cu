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
// second walks a portion's chunks in order: a warp keeps 16 value columns of S^T in its accumulators from the portion's first
// chunk to its last; as the first operand of the products with Q and W, and with U^T as the first operand of the products with
// P and K, the accumulators' own layout is that of the operand, so the state never leaves the registers. The next two
// chunks' records travel to shared memory meanwhile (cp.async).
#include "attn_mma.cuh"
#include <math.h>

namespace {
using namespace fzattn;
constexpr int C = 16;                       // tokens per chunk
constexpr int COOK_THREADS = 256;
constexpr int WARPS = 4;                    // warps of the second kernel: 16 value columns each
constexpr int STAGES = 3;
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

// The record of a (chunk, head), in bytes: MATS matrices [16][dkp] of bf16 (Q, K and for the delta rule W; rounding, then
// rest), P [16][16] (rounding, rest), the decays of the chunk (dkp floats), V: rounding and rest [16][dvp] bf16 (linear
// attention) or V' [16][dvp] float (delta rule).
struct Record {
  int dkp, dvp, mats;
  __host__ __device__ Record(int dkp_, int dv, bool delta) : dkp(dkp_), dvp((dv + 15) / 16 * 16), mats(delta ? 6 : 4) {}
  __host__ __device__ int mat() const { return C * dkp * 2; }
  __host__ __device__ int p() const { return mats * mat(); }
  __host__ __device__ int decay() const { return p() + 2 * C * C * 2; }
  __host__ __device__ int v() const { return decay() + dkp * 4; }
  __host__ __device__ long long bytes() const { return v() + C * dvp * 4; }
};
// The records of a portion that begins at row r stand from place ceil(r / 8) on. A portion of n >= 16 rows has ceil(n / 16) of
// them, and ceil((r + n) / 8) >= ceil(r / 8) + ceil((n - 7) / 8) >= ceil(r / 8) + ceil(n / 16): no two portions of 16 rows and
// more share a place, and a step of N rows needs ceil(N / 8) places, whatever portions it holds.
__device__ __forceinline__ long long record_place(int row0, int chunk) { return (row0 + 7) / 8 + chunk; }

// A [16][cols] matrix of shared memory (ld floats per row) times row factors, as rounding and rest.
template <typename Fn>
__device__ __forceinline__ void leave_matrix(unsigned char* hi, unsigned char* lo, int cols, Fn value) {
  for (int e = threadIdx.x; e < C * cols / 2; e += COOK_THREADS) {
    const int t = e / (cols / 2), c = 2 * (e - t * (cols / 2));
    uint32_t h, l;
    split2(value(t, c), value(t, c + 1), h, l);
    ((uint32_t*)hi)[e] = h;
    ((uint32_t*)lo)[e] = l;
  }
}

struct CookArgs {
  const int* seg;
  int H, Hk, dk, dv, dkp, min_rows;
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
__global__ void __launch_bounds__(COOK_THREADS)
gla_cook_kernel(const CookArgs a) {
  fz_grid_launch_dependents();
  const int s = blockIdx.x, c0 = blockIdx.y * C, h = blockIdx.z;
  const int row0 = a.seg[4 * s], cnt = a.seg[4 * s + 1], slot = a.seg[4 * s + 3];
  fz_grid_wait();
  if (cnt < a.min_rows || c0 >= cnt || slot < 0) return;
  extern __shared__ __align__(16) float sm[];
  const int dk = a.dk, dkp = a.dkp, LD = dkp + 1, valid = min(C, cnt - c0);
  float* q = sm;                 // [16][LD]
  float* k = q + C * LD;
  float* L = k + C * LD;         // logarithms (base 2) of the decays, then their running sums
  const Record rec(dkp, a.dv, false);
  unsigned char* out = a.scratch + (record_place(row0, blockIdx.y) * a.H + h) * rec.bytes();
  const size_t n0 = (size_t)(row0 + c0);
  for (int e = threadIdx.x; e < C * dkp; e += COOK_THREADS) {
    const int t = e / dkp, c = e - t * dkp;
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
  {                              // V needs nothing of the above
    unsigned char* v = out + rec.v();
    leave_matrix(v, v + C * rec.dvp * 2, rec.dvp, [&](int t, int c) {
      return t < valid && c < a.dv ? a.proj[(n0 + t) * a.ld + (size_t)2 * a.H * dk + (size_t)h * a.dv + c] : 0.f;
    });
  }
  __syncthreads();
  if (threadIdx.x < dkp) {
    float run = 0.f;
#pragma unroll
    for (int t = 0; t < C; ++t) { run += L[t * LD + threadIdx.x]; L[t * LD + threadIdx.x] = run; }
    ((float*)(out + rec.decay()))[threadIdx.x] = ex2(run);
  }
  __syncthreads();
  leave_matrix(out, out + rec.mat(), dkp, [&](int t, int c) { return q[t * LD + c] * ex2(L[t * LD + c]); });
  leave_matrix(out + 2 * rec.mat(), out + 3 * rec.mat(), dkp, [&](int t, int c) { return k[t * LD + c] * ex2(L[(C - 1) * LD + c] - L[t * LD + c]); });
  __nv_bfloat16* P = (__nv_bfloat16*)(out + rec.p());
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int half = 0; half < 2; ++half) {         // a warp takes token `warp` and token 15 - `warp`: 17 pairs
    const int t = half == 0 ? warp : C - 1 - warp;
    float qt[4], Lt[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = lane + 32 * i;
      qt[i] = c < dkp ? q[t * LD + c] : 0.f;
      Lt[i] = c < dkp ? L[t * LD + c] : 0.f;
    }
    float mine = 0.f;                            // lane s keeps P_ts
    for (int x = 0; x <= t; ++x) {
      float acc = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int c = lane + 32 * i;
        if (c < dkp) acc = fmaf(qt[i] * k[x * LD + c], ex2(Lt[i] - L[x * LD + c]), acc);
      }
      acc = warp_sum(acc);
      if (lane == x) mine = acc;
    }
    if (lane < C) {
      const __nv_bfloat16 hi = __float2bfloat16_rn(mine);
      P[t * C + lane] = hi;
      P[C * C + t * C + lane] = __float2bfloat16_rn(mine - __bfloat162float(hi));
    }
  }
}

__global__ void __launch_bounds__(COOK_THREADS)
delta_cook_kernel(const CookArgs a) {
  fz_grid_launch_dependents();
  const int s = blockIdx.x, c0 = blockIdx.y * C, h = blockIdx.z;
  const int row0 = a.seg[4 * s], cnt = a.seg[4 * s + 1], slot = a.seg[4 * s + 3];
  const float rate2 = expf(a.a_log[h]) * LOG2E, bias = a.dt_bias[h];
  fz_grid_wait();
  if (cnt < a.min_rows || c0 >= cnt || slot < 0) return;
  extern __shared__ __align__(16) float sm[];
  const int dk = a.dk, dkp = a.dkp, LD = dkp + 1, valid = min(C, cnt - c0);
  const Record rec(dkp, a.dv, true);
  const int dvp = rec.dvp;
  float* q = sm;                 // [16][LD]
  float* k = q + C * LD;
  float* v = k + C * LD;         // [16][dvp]
  float* M = v + C * dvp;        // [16][17]: beta_t e^{L_t - L_s} k_t . k_s below the diagonal
  float* T1 = M + C * 17;        // [16][17]: T diag(beta)
  float* T2 = T1 + C * 17;       // [16][17]: T diag(beta e^L)
  float* L = T2 + C * 17;        // [16]
  float* b = L + C;              // [16]
  unsigned char* out = a.scratch + (record_place(row0, blockIdx.y) * a.H + h) * rec.bytes();
  const size_t n0 = (size_t)(row0 + c0);
  const int kh = h / (a.H / a.Hk), W = 2 * a.Hk * dk + a.H * a.dv;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int half = 0; half < 2; ++half) {         // a warp brings two tokens in: unit vectors
    const int t = warp + 8 * half;
    const __nv_bfloat16* in = a.qkv + (n0 + t) * W;
    float qv[4], kv[4], sq = 0.f, sk = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = lane + 32 * i;
      const bool ok = c < dk && t < valid;
      qv[i] = ok ? __bfloat162float(in[(size_t)kh * dk + c]) : 0.f;
      kv[i] = ok ? __bfloat162float(in[(size_t)(a.Hk + kh) * dk + c]) : 0.f;
      sq = fmaf(qv[i], qv[i], sq);
      sk = fmaf(kv[i], kv[i], sk);
    }
    const float nq = sqrtf(warp_sum(sq) + a.unit_eps), nk = sqrtf(warp_sum(sk) + a.unit_eps);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = lane + 32 * i;
      if (c < dkp) {
        q[t * LD + c] = __fmul_rn(__fdiv_rn(qv[i], nq), a.q_scale);
        k[t * LD + c] = __fdiv_rn(kv[i], nk);
      }
    }
  }
  for (int e = threadIdx.x; e < C * dvp; e += COOK_THREADS) {
    const int t = e / dvp, c = e - t * dvp;
    v[e] = t < valid && c < a.dv ? __bfloat162float(a.qkv[(n0 + t) * W + (size_t)2 * a.Hk * dk + (size_t)h * a.dv + c]) : 0.f;
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
  __nv_bfloat16* P = (__nv_bfloat16*)(out + rec.p());
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = half == 0 ? warp : C - 1 - warp;
    float qt[4], kt[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = lane + 32 * i;
      qt[i] = c < dkp ? q[t * LD + c] : 0.f;
      kt[i] = c < dkp ? k[t * LD + c] : 0.f;
    }
    float qk = 0.f, kk = 0.f;                    // lane s keeps the products with k_s
    for (int x = 0; x <= t; ++x) {
      float p = 0.f, m = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int c = lane + 32 * i;
        const float kx = c < dkp ? k[x * LD + c] : 0.f;
        p = fmaf(qt[i], kx, p);
        m = fmaf(kt[i], kx, m);
      }
      p = warp_sum(p);
      m = warp_sum(m);
      if (lane == x) { qk = p; kk = m; }
    }
    if (lane < C) {
      const float f = lane <= t ? ex2(L[t] - L[lane]) : 0.f;
      qk *= f;
      const __nv_bfloat16 hi = __float2bfloat16_rn(qk);
      P[t * C + lane] = hi;
      P[C * C + t * C + lane] = __float2bfloat16_rn(qk - __bfloat162float(hi));
      M[t * 17 + lane] = lane < t ? b[t] * f * kk : 0.f;
    }
  }
  __syncthreads();
  if (threadIdx.x < C) {                         // column j of T by substitution: T_tj = [t = j] - sum_{s < t} M_ts T_sj
    const int j = threadIdx.x;
    float x[C];
#pragma unroll
    for (int t = 0; t < C; ++t) {
      float acc = t == j ? 1.f : 0.f;
#pragma unroll
      for (int y = 0; y < t; ++y) acc = fmaf(-M[t * 17 + y], x[y], acc);
      x[t] = acc;
    }
    const float b1 = b[j], b2 = b1 * ex2(L[j]);
#pragma unroll
    for (int t = 0; t < C; ++t) { T1[t * 17 + j] = x[t] * b1; T2[t * 17 + j] = x[t] * b2; }
  }
  const float last = L[C - 1];
  leave_matrix(out, out + rec.mat(), dkp, [&](int t, int c) { return q[t * LD + c] * ex2(L[t]); });
  leave_matrix(out + 2 * rec.mat(), out + 3 * rec.mat(), dkp, [&](int t, int c) { return k[t * LD + c] * ex2(last - L[t]); });
  if (threadIdx.x < dkp) ((float*)(out + rec.decay()))[threadIdx.x] = ex2(last);
  __syncthreads();
  leave_matrix(out + 4 * rec.mat(), out + 5 * rec.mat(), dkp, [&](int t, int c) {
    float acc = 0.f;
    for (int y = 0; y <= t; ++y) acc = fmaf(T2[t * 17 + y], k[y * LD + c], acc);
    return acc;
  });
  float* vout = (float*)(out + rec.v());
  for (int e = threadIdx.x; e < C * dvp; e += COOK_THREADS) {
    const int t = e / dvp, c = e - t * dvp;
    float acc = 0.f;
    for (int y = 0; y <= t; ++y) acc = fmaf(T1[t * 17 + y], v[y * dvp + c], acc);
    vout[e] = acc;
  }
}

// ---- the second kernel: grid (portions, heads, blocks of 64 value columns)
// A stage of shared memory: the record's matrices with rows of dkp + 8 values, P with rows of 24, the decays, this block's 64
// columns of V with rows of 72 bf16 (rounding, rest) or 68 floats (an odd number of 16-byte units per row: no bank conflicts).
template <int DKP, bool DELTA> struct Stage {
  static constexpr int MATS = DELTA ? 6 : 4, ROW = DKP * 2 + 16, MAT = C * ROW, P_ROW = 48, P_MAT = C * P_ROW;
  static constexpr int P = MATS * MAT, DECAY = P + 2 * P_MAT, V = DECAY + DKP * 4;
  static constexpr int V_ROW = DELTA ? 272 : 144, V_MAT = C * V_ROW, BYTES = V + (DELTA ? 1 : 2) * V_MAT;
};

template <int DKP, bool DELTA>
__global__ void __launch_bounds__(32 * WARPS)
scan_chunk_kernel(const unsigned char* __restrict__ scratch, int H, int dv, float* __restrict__ state, const int* __restrict__ seg,
                  int min_rows, float* __restrict__ out) {
  using St = Stage<DKP, DELTA>;
  fz_grid_launch_dependents();
  const int s = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * 16 * WARPS;
  const int row0 = seg[4 * s], cnt = seg[4 * s + 1], slot = seg[4 * s + 3];
  fz_grid_wait();
  if (cnt < min_rows || cnt <= 0 || slot < 0) return;
  extern __shared__ __align__(128) unsigned char smem[];
  const uint32_t s0 = smem_u32(smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, q2 = 2 * (lane & 3);            // an accumulator's row (and row + 8) and first column
  const Record rec(DKP, dv, DELTA);
  const int nc = (cnt + C - 1) / C;
  const unsigned char* base = scratch + (record_place(row0, 0) * H + h) * rec.bytes();
  const long long step = (long long)H * rec.bytes();
  const int vcols = min(16 * WARPS, rec.dvp - col0);       // this block's columns of V (a multiple of 16)

  auto issue = [&](int c) {
    if (c < nc) {
      const unsigned char* r = base + c * step;
      const uint32_t st = s0 + (c % STAGES) * St::BYTES;
      constexpr int PER = DKP / 8;                         // 16-byte pieces per row
      for (int e = tid; e < St::MATS * C * PER; e += 32 * WARPS) cp_async16(st + (e / PER) * St::ROW + (e % PER) * 16, r + e * 16, true);
      for (int e = tid; e < 2 * C * 2; e += 32 * WARPS) cp_async16(st + St::P + (e >> 1) * St::P_ROW + (e & 1) * 16, r + rec.p() + e * 16, true);
      if (tid < DKP / 4) cp_async16(st + St::DECAY + tid * 16, r + rec.decay() + tid * 16, true);
      const int rows = DELTA ? C : 2 * C, per = DELTA ? vcols / 4 : vcols / 8, src = rec.dvp * (DELTA ? 4 : 2), at = col0 * (DELTA ? 4 : 2);
      for (int e = tid; e < rows * per; e += 32 * WARPS) {
        const int t = e / per, i = e - t * per;
        cp_async16(st + St::V + t * St::V_ROW + i * 16, r + rec.v() + (long long)t * src + at + i * 16, true);
      }
    }
    cp_async_commit();                                     // (an empty group past the last chunk keeps the count)
  };
#pragma unroll
  for (int c = 0; c < STAGES - 1; ++c) issue(c);

  constexpr int KN = DKP / 16;
  float S[2 * KN][4];                                      // S^T: rows are value columns, columns are key channels
  const int ca = col0 + 16 * warp + g, cb = ca + 8;        // this thread's two value columns
  float* sa = state + (((size_t)slot * H + h) * dv + ca) * DKP + q2;
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
  const bool mine = 16 * warp < vcols;

  for (int c = 0; c < nc; ++c) {
    cp_async_wait<STAGES - 2>();
    __syncthreads();
    issue(c + STAGES - 1);                                 // into the place of chunk c - 1
    if (!mine) continue;
    const uint32_t st = s0 + (c % STAGES) * St::BYTES;
    const unsigned char* sp = smem + (c % STAGES) * St::BYTES;
    float O[3][2][4], D[DELTA ? 3 : 1][2][4];              // hi . hi, rest . hi, hi . rest
#pragma unroll
    for (int x = 0; x < 3; ++x)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) { O[x][n][e] = 0.f; if (DELTA) D[DELTA ? x : 0][n][e] = 0.f; }
    const uint32_t a_q = st + off_n * St::ROW + (mi & 1) * 16;
#pragma unroll
    for (int k = 0; k < KN; ++k) {
      uint32_t hi[4], lo[4];
      split2(S[2 * k][0], S[2 * k][1], hi[0], lo[0]);
      split2(S[2 * k][2], S[2 * k][3], hi[1], lo[1]);
      split2(S[2 * k + 1][0], S[2 * k + 1][1], hi[2], lo[2]);
      split2(S[2 * k + 1][2], S[2 * k + 1][3], hi[3], lo[3]);
      uint32_t bh[4], bl[4];
      ldmatrix_x4(bh, a_q + 32 * k);
      ldmatrix_x4(bl, a_q + St::MAT + 32 * k);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        mma_bf16(O[0][n], hi, bh[2 * n], bh[2 * n + 1]);
        mma_bf16(O[1][n], lo, bh[2 * n], bh[2 * n + 1]);
        mma_bf16(O[2][n], hi, bl[2 * n], bl[2 * n + 1]);
      }
      if constexpr (DELTA) {
        ldmatrix_x4(bh, a_q + 4 * St::MAT + 32 * k);
        ldmatrix_x4(bl, a_q + 5 * St::MAT + 32 * k);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          mma_bf16(D[0][n], hi, bh[2 * n], bh[2 * n + 1]);
          mma_bf16(D[1][n], lo, bh[2 * n], bh[2 * n + 1]);
          mma_bf16(D[2][n], hi, bl[2 * n], bl[2 * n + 1]);
        }
      }
    }
    uint32_t uh[4], ul[4];                                 // U^T (value columns x tokens) as a first operand
    if constexpr (DELTA) {
      const float* v = (const float*)(sp + St::V) + 16 * warp + g;
      constexpr int VR = St::V_ROW / 4;
      float U[2][4];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          U[n][e] = v[(8 * n + q2 + (e & 1)) * VR + (e >> 1) * 8] - (D[0][n][e] + (D[1][n][e] + D[2][n][e]));
      split2(U[0][0], U[0][1], uh[0], ul[0]);
      split2(U[0][2], U[0][3], uh[1], ul[1]);
      split2(U[1][0], U[1][1], uh[2], ul[2]);
      split2(U[1][2], U[1][3], uh[3], ul[3]);
    } else {
      const uint32_t a_v = st + St::V + off_n * St::V_ROW + (16 * warp + (mi & 1) * 8) * 2;
      ldmatrix_x4_trans(uh, a_v);
      ldmatrix_x4_trans(ul, a_v + St::V_MAT);
    }
    {
      const uint32_t a_p = st + St::P + off_n * St::P_ROW + (mi & 1) * 16;
      uint32_t bh[4], bl[4];
      ldmatrix_x4(bh, a_p);
      ldmatrix_x4(bl, a_p + St::P_MAT);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        mma_bf16(O[0][n], uh, bh[2 * n], bh[2 * n + 1]);
        mma_bf16(O[1][n], ul, bh[2 * n], bh[2 * n + 1]);
        mma_bf16(O[2][n], uh, bl[2 * n], bl[2 * n + 1]);
      }
    }
    const uint32_t a_k = st + 2 * St::MAT + off_k * St::ROW + (mi >> 1) * 16;
    const float* dec = (const float*)(sp + St::DECAY) + q2;
#pragma unroll
    for (int k = 0; k < KN; ++k) {
      uint32_t bh[4], bl[4];
      ldmatrix_x4_trans(bh, a_k + 32 * k);
      ldmatrix_x4_trans(bl, a_k + St::MAT + 32 * k);
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
    const int valid = min(C, cnt - c * C);
    float* dst = out + ((size_t)(row0 + c * C) * H + h) * dv;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = 8 * n + q2 + (e & 1), col = e < 2 ? ca : cb;
        if (t < valid && col < dv) dst[(size_t)t * H * dv + col] = O[0][n][e] + (O[1][n][e] + O[2][n][e]);
      }
  }
  cp_async_wait<0>();
  if (!mine) return;
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
int launch_scan(const CookArgs& a, float* state, int n_seg, float* out, cudaStream_t stream) {
  constexpr size_t smem = (size_t)STAGES * Stage<DKP, DELTA>::BYTES;
  static size_t allowed = 48 * 1024;
  int st = allow_smem(scan_chunk_kernel<DKP, DELTA>, smem, allowed);
  if (st != FZ_OK) return st;
  fz_launch(scan_chunk_kernel<DKP, DELTA>, dim3(n_seg, a.H, (a.dv + 16 * WARPS - 1) / (16 * WARPS)), dim3(32 * WARPS), smem, stream,
            (const unsigned char*)a.scratch, a.H, a.dv, state, a.seg, a.min_rows, out);
  FZ_LAUNCH_CHECK();
  return FZ_OK;
}

template <bool DELTA>
int run(CookArgs a, float* state, int n_seg, int max_rows, float* out, cudaStream_t stream) {
  a.dkp = padded_keys(a.dk);
  const int chunks = (max_rows + C - 1) / C, LD = a.dkp + 1;
  if (chunks > 65535) return FZ_TOO_LARGE;
  const Record rec(a.dkp, a.dv, DELTA);
  const size_t smem = sizeof(float) * (DELTA ? 2 * (size_t)C * LD + (size_t)C * rec.dvp + 3 * C * 17 + 2 * C : 3 * (size_t)C * LD);
  static size_t allowed = 48 * 1024;
  auto cook = DELTA ? delta_cook_kernel : gla_cook_kernel;
  int st = allow_smem(cook, smem, allowed);
  if (st != FZ_OK) return st;
  fz_launch(cook, dim3(n_seg, chunks, a.H), dim3(COOK_THREADS), smem, stream, a);
  FZ_LAUNCH_CHECK();
  switch (a.dkp) {
    case 16: return launch_scan<16, DELTA>(a, state, n_seg, out, stream);
    case 32: return launch_scan<32, DELTA>(a, state, n_seg, out, stream);
    case 64: return launch_scan<64, DELTA>(a, state, n_seg, out, stream);
    default: return launch_scan<128, DELTA>(a, state, n_seg, out, stream);
  }
}
}  // namespace

// Sizes taken: keys of 9 to 128, values of up to 1,024.
FZ_API int fz_scan_chunk_check(int H, int dk, int dv) {
  return (H > 0 && H <= 65535 && dk > 8 && dk <= 128 && dv > 0 && dv <= 1024) ? FZ_OK : FZ_BAD_SHAPE;
}

// Bytes of scratch for a step of N rows (see record_place).
FZ_API long long fz_scan_chunk_scratch(int N, int H, int dk, int dv, int delta) {
  return ((long long)N / 8 + 1) * H * Record(padded_keys(dk), dv, delta != 0).bytes();
}

// Portions of min_rows rows and more (max_rows at most); the state is (slots, H, dv, padded keys). See fz_channel_decay_scan.
FZ_API int fz_gla_chunk(const float* proj, int ld, int H, int dk, int dv, const float* z, float inv_root, float q_scale, float* state,
                        const int* seg, int n_seg, int min_rows, int max_rows, void* scratch, float* out, cudaStream_t stream) {
  if (n_seg <= 0) return FZ_OK;
  if (fz_scan_chunk_check(H, dk, dv) != FZ_OK || ld < H * (2 * dk + dv) || scratch == nullptr || ((uintptr_t)scratch & 15) || min_rows < C) return FZ_BAD_SHAPE;
  CookArgs a = {};
  a.seg = seg; a.H = a.Hk = H; a.dk = dk; a.dv = dv; a.min_rows = min_rows; a.scratch = (unsigned char*)scratch;
  a.proj = proj; a.ld = ld; a.z = z; a.inv_root = inv_root; a.q_scale = q_scale;
  return run<false>(a, state, n_seg, max_rows, out, stream);
}

// See fz_gated_delta_scan (one decay per head).
FZ_API int fz_delta_chunk(const void* qkv, int H, int Hk, int dk, int dv, const float* high, int ldh, const float* beta, int ldb,
                          const float* a_log, const float* dt_bias, float unit_eps, float q_scale, float* state, const int* seg,
                          int n_seg, int min_rows, int max_rows, void* scratch, float* out, cudaStream_t stream) {
  if (n_seg <= 0) return FZ_OK;
  if (fz_scan_chunk_check(H, dk, dv) != FZ_OK || Hk <= 0 || H % Hk || scratch == nullptr || ((uintptr_t)scratch & 15) || min_rows < C) return FZ_BAD_SHAPE;
  CookArgs a = {};
  a.seg = seg; a.H = H; a.Hk = Hk; a.dk = dk; a.dv = dv; a.min_rows = min_rows; a.scratch = (unsigned char*)scratch;
  a.qkv = (const __nv_bfloat16*)qkv; a.high = high; a.ldh = ldh; a.beta = beta; a.ldb = ldb; a.a_log = a_log; a.dt_bias = dt_bias;
  a.unit_eps = unit_eps; a.q_scale = q_scale;
  return run<true>(a, state, n_seg, max_rows, out, stream);
}

#ifdef FZ_TIMELINE
FZ_TIMELINE_READER(scan_chunk)
#endif
