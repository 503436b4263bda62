// The selective state space scan of long portions in bfloat16, 64 tokens at a time on tensor cores (mma.sync m16n8k16).
// With d_t = softplus(dt + bias), L_t = sum of -exp(A) d over the chunk's tokens up to t, and M the state before the chunk,
//
//   y_t = exp(L_t) C_t^T M + sum_{s <= t} (C_t . B_s) exp(L_t - L_s) d_s x_s + D x_t
//   M  <- exp(L_last) M + sum_s B_s (exp(L_last - L_s) d_s x_s)^T
//
// which is the token-by-token recurrence of ssd.cu in another order. x, B and C are bfloat16 as they come; everything else
// is 32-bit: the decays, the sums, the state (float32 accumulators that stay in registers from the portion's first chunk to
// its last). Where a 32-bit value is an operand of a product (the state, the weighted C . B, the weighted x) it goes in as
// the sum of two bfloat16 numbers, its rounding and the rounding of what is left, and both are multiplied: a relative
// error of 2^-17 per term.
//
// A block owns PB value columns of one head of one portion. Eight warps compute the results of a chunk: a warp takes 16
// tokens and half of what they need, first every second 16 x 16 tile of the weighted C . B (left in shared memory as
// operands), then half of the value columns. Eight others compute the state after the chunk: first the weighted x (left in
// shared memory as operands), then units of 16 state rows x 16 columns, which they leave as operands for the next chunk's
// results, and bring the rows of the next one or two chunks in (cp.async; bulk copies of a row each took twice as long as the
// arithmetic). One more warp computes the next chunk's decays. Each group of eight has a barrier between its two halves,
// the block one per chunk.
#include "attn_mma.cuh"
#include <math.h>

namespace {
using namespace fzattn;
constexpr int Q = 64;                       // tokens per chunk
constexpr int SSD_THREADS = 544;        // eight warps for the results, eight for the state, one for the decays
constexpr float LOG2E = 1.4426950408889634f;

// 2^x for x <= 0 (results below the normal range are zero)
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void group_barrier(int id) { asm volatile("bar.sync %0, 256;" ::"r"(id) : "memory"); }
__device__ __forceinline__ float softplus32(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// Two 32-bit values as bfloat16 pairs: their roundings, and the roundings of what is left.
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  hi = *(const uint32_t*)&h;
  lo = pack_bf16(a - f.x, b - f.y);
}
__device__ __forceinline__ float2 unpack2(uint32_t v) { return __bfloat1622float2(*(const __nv_bfloat162*)&v); }

struct SsdChunkArgs {
  const __nv_bfloat16* xbc;                 // rows of W values: [x (H P) | B (G N) | C (G N)]
  int W, H, G, N, P;
  const float* dt;
  int ldt, off_dt;
  const float *dt_bias, *a_log, *skip;
  float* state;                             // (slots, H, P, npad)
  int npad;
  const int* seg;
  int min_rows;                             // portions of fewer rows are left to the other kernel
  float* out;                               // (rows, H P)
};

__host__ __device__ constexpr int pad_units(int n) { return n + 8; }      // an odd number of 16-byte units per row: no bank conflicts

// PB: value columns per block (16 or 32). UM: units of 16 state rows x 16 columns per warp (1 or 2). ST: chunks in shared
// memory at a time (3, or 2 where three do not fit). grid (portions, heads, P / PB).
template <int PB, int UM, int ST>
__global__ void __launch_bounds__(SSD_THREADS)
ssd_chunk_kernel(const SsdChunkArgs p) {
  fz_grid_launch_dependents();
  const int s = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * PB;
  const int row0 = p.seg[4 * s], cnt = p.seg[4 * s + 1], slot = p.seg[4 * s + 3];
  const float rate2 = expf(p.a_log[h]) * LOG2E, bias = p.dt_bias[h], D = p.skip[h];
  fz_grid_wait();
  if (cnt < p.min_rows || cnt <= 0 || slot < 0) return;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int N = p.N, KN = N >> 4, SN = pad_units(N);
  constexpr int SP = pad_units(PB), SQ = pad_units(Q), NT = PB / 16;      // NT: 8-column tiles per result warp
  __nv_bfloat16* Cs = (__nv_bfloat16*)smem_raw;            // [ST][Q][SN]
  __nv_bfloat16* Bs = Cs + ST * Q * SN;                    // [ST][Q][SN]
  __nv_bfloat16* Xs = Bs + ST * Q * SN;                    // [ST][Q][SP]
  __nv_bfloat16* Ms = Xs + ST * Q * SP;                    // [2][2][N][SP]: the state before a chunk, rounding and rest
  __nv_bfloat16* Gs = Ms + 4 * N * SP;                     // [2][Q][SQ]: the weighted C . B, rounding and rest
  __nv_bfloat16* Ws = Gs + 2 * Q * SQ;                     // [2][Q][SP]: the weighted x, rounding and rest
  float* scal = (float*)(Ws + 2 * Q * SP);                 // [2][4][Q]: L in powers of two, exp(L), d, exp(L_last - L) d
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = lane >> 2, q2 = (lane & 3) * 2;           // an accumulator's row (and row + 8) and first column
  const int g = h / (p.H / p.G);
  const int nc = (cnt + Q - 1) / Q;
  const size_t off_x = (size_t)h * p.P + p0, off_b = (size_t)p.H * p.P + (size_t)g * N, off_c = off_b + (size_t)p.G * N;

  const int per = KN >= 8 ? 3 : 2;           // 2^per threads side by side on a token's run of B or C
  auto load_chunk = [&](int c) {                           // by the state's warps; past the portion's end: zeros
    if (c < nc) {
      const int st = c % ST, me = tid & 255;
      const __nv_bfloat16* in = p.xbc + (size_t)(row0 + c * Q) * p.W;
      for (int r = me >> per; r < Q; r += 256 >> per) {
        const bool ok = c * Q + r < cnt;
        const __nv_bfloat16* row = in + (ok ? (size_t)r * p.W : 0);
        const uint32_t at = (uint32_t)((st * Q + r) * SN * 2);
        for (int j = me & ((1 << per) - 1); j < 2 * KN; j += 1 << per) {
          cp_async16(smem_u32(Cs) + at + 16 * j, row + off_c + 8 * j, ok);
          cp_async16(smem_u32(Bs) + at + 16 * j, row + off_b + 8 * j, ok);
        }
      }
      const int r = me >> 2;
      const bool ok = c * Q + r < cnt;
      if ((me & 3) < PB / 8)
        cp_async16(smem_u32(Xs + (st * Q + r) * SP) + 16 * (me & 3), in + (ok ? (size_t)r * p.W : 0) + off_x + 8 * (me & 3), ok);
    }
    cp_async_commit();                                     // (an empty group past the last chunk keeps the count)
  };
  // the scalars of a chunk, two tokens per lane of one warp; r0, r1: the tokens' raw step sizes
  auto raw_steps = [&](int c, float& r0, float& r1) {
    const int t = c * Q + 2 * lane;
    r0 = t < cnt ? p.dt[(size_t)(row0 + t) * p.ldt + p.off_dt + h] : 0.f;
    r1 = t + 1 < cnt ? p.dt[(size_t)(row0 + t + 1) * p.ldt + p.off_dt + h] : 0.f;
  };
  auto scalars = [&](int c, float r0, float r1) {
    const int t = c * Q + 2 * lane;
    const float d0 = t < cnt ? softplus32(r0 + bias) : 0.f, d1 = t + 1 < cnt ? softplus32(r1 + bias) : 0.f;
    const float a0 = -rate2 * d0, a1 = -rate2 * d1;
    float incl = a0 + a1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += v;
    }
    float before = __shfl_up_sync(0xffffffffu, incl, 1);
    if (lane == 0) before = 0.f;
    const float last = __shfl_sync(0xffffffffu, incl, 31);
    const float l0 = before + a0, l1 = incl;
    float* sc = scal + (c & 1) * 4 * Q + 2 * lane;
    *(float2*)sc = make_float2(l0, l1);
    *(float2*)(sc + Q) = make_float2(ex2(l0), ex2(l1));
    *(float2*)(sc + 2 * Q) = make_float2(d0, d1);
    *(float2*)(sc + 3 * Q) = make_float2(ex2(last - l0) * d0, ex2(last - l1) * d1);
  };

  // of the warps that keep the state: units sw, sw + 8; unit u: state rows 16 (u % KN), columns 16 (u / KN)
  const int sw = warp - 8;
  int ur[UM], uc[UM];
  bool own[UM];
#pragma unroll
  for (int i = 0; i < UM; ++i) {
    const int u = max(sw, 0) + 8 * i;
    own[i] = u < KN * NT;
    ur[i] = 16 * (u % KN);
    uc[i] = 16 * (u / KN);
  }
  float S[UM][2][4];
  auto leave_state = [&](int buf) {
    __nv_bfloat16* hi = Ms + (size_t)buf * 2 * N * SP;
    __nv_bfloat16* lo = hi + (size_t)N * SP;
#pragma unroll
    for (int i = 0; i < UM; ++i) {
      if (!own[i]) break;
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int at = (ur[i] + gq) * SP + uc[i] + 8 * n + q2;
        uint32_t a, b;
        split2(S[i][n][0], S[i][n][1], a, b);
        *(uint32_t*)(hi + at) = a; *(uint32_t*)(lo + at) = b;
        split2(S[i][n][2], S[i][n][3], a, b);
        *(uint32_t*)(hi + at + 8 * SP) = a; *(uint32_t*)(lo + at + 8 * SP) = b;
      }
    }
  };
  float* sp = p.state + (((size_t)slot * p.H + h) * p.P + p0) * p.npad;
  auto state_at = [&](int i, int n, int e) {
    return (size_t)(uc[i] + 8 * n + q2 + (e & 1)) * p.npad + ur[i] + gq + (e & 2) * 4;
  };

  if (sw == 8) {                                           // the warp that computes the decays
    float r0, r1;
    raw_steps(0, r0, r1);
    scalars(0, r0, r1);
    raw_steps(1, r0, r1);                                  // (zeros past the end)
    __syncthreads();
    for (int c = 0; c < nc; ++c) {
      if (c + 1 < nc) {
        const float n0 = r0, n1 = r1;
        raw_steps(c + 2, r0, r1);
        scalars(c + 1, n0, n1);
      }
      __syncthreads();
    }
    return;
  }
  if (sw >= 0) {
#pragma unroll
    for (int c = 0; c < ST - 1; ++c) load_chunk(c);
#pragma unroll
    for (int i = 0; i < UM; ++i)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][n][e] = own[i] ? sp[state_at(i, n, e)] : 0.f;
    leave_state(0);
    cp_async_wait<ST - 2>();
  }
  __syncthreads();

  for (int c = 0; c < nc; ++c) {
    const int st = c & 1, valid = min(Q, cnt - c * Q);
    const bool more = c + 1 < nc;
    const int slot_in = c % ST;
    const __nv_bfloat16* Cc = Cs + slot_in * Q * SN;
    const __nv_bfloat16* Bc = Bs + slot_in * Q * SN;
    const __nv_bfloat16* Xc = Xs + slot_in * Q * SP;
    const float* sc = scal + st * 4 * Q;
    if (sw < 0) {
      const int rt = warp >> 1, half = warp & 1;           // 16 tokens; which tiles and which columns
      const bool live = 16 * rt < valid;
      const int ta = 16 * rt + gq, tb = ta + 8;            // this thread's two tokens
      float Y[NT][4], Z[NT][4];                            // products with the roundings and with the rests
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) Y[n][e] = Z[n][e] = 0.f;
      if (live) {
        float G[2][2][4];                                  // tiles half and half + 2
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int e = 0; e < 4; ++e) G[i][u][e] = 0.f;
        const uint32_t ac = smem_u32(Cc + (16 * rt + (lane & 15)) * SN + 8 * (lane >> 4));
        const uint32_t ab = smem_u32(Bc + (16 * half + ((lane >> 4) << 3) + (lane & 7)) * SN + 8 * ((lane >> 3) & 1));
        // the state's rounding and rest in one load: lanes 0 .. 15 the rounding's rows, 16 .. 31 the rest's
        const uint32_t am = smem_u32(Ms + ((size_t)st * 2 + (lane >> 4)) * N * SP + (lane & 15) * SP + 8 * NT * half);
#pragma unroll 4
        for (int k = 0; k < KN; ++k) {
          uint32_t a[4], b[4];
          ldmatrix_x4(a, ac + 32 * k);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            if (half + 2 * i > rt) break;                  // tokens after this warp's: not seen
            ldmatrix_x4(b, ab + (32 * i * SN) * 2 + 32 * k);
            mma_bf16(G[i][0], a, b[0], b[1]);
            mma_bf16(G[i][1], a, b[2], b[3]);
          }
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            ldmatrix_x4_trans(b, am + (16 * k * SP) * 2 + 16 * n);
            mma_bf16(Y[n], a, b[0], b[1]);
            mma_bf16(Z[n], a, b[2], b[3]);
          }
        }
        const float la = sc[ta], lb = sc[tb], ea = sc[Q + ta], eb = sc[Q + tb];
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          Y[n][0] *= ea; Y[n][1] *= ea; Y[n][2] *= eb; Y[n][3] *= eb;
          Z[n][0] *= ea; Z[n][1] *= ea; Z[n][2] *= eb; Z[n][3] *= eb;
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int j = half + 2 * i;
          if (j > rt) break;
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const int t = 16 * j + 8 * u + q2;             // the earlier tokens of this thread's columns: t, t + 1
            const float2 l = *(const float2*)(sc + t), d = *(const float2*)(sc + 2 * Q + t);
            const float* w = G[i][u];
            const float w0 = t <= ta ? w[0] * (ex2(la - l.x) * d.x) : 0.f, w1 = t + 1 <= ta ? w[1] * (ex2(la - l.y) * d.y) : 0.f;
            const float w2 = t <= tb ? w[2] * (ex2(lb - l.x) * d.x) : 0.f, w3 = t + 1 <= tb ? w[3] * (ex2(lb - l.y) * d.y) : 0.f;
            uint32_t hi, lo;
            split2(w0, w1, hi, lo);
            *(uint32_t*)(Gs + ta * SQ + t) = hi; *(uint32_t*)(Gs + (Q + ta) * SQ + t) = lo;
            split2(w2, w3, hi, lo);
            *(uint32_t*)(Gs + tb * SQ + t) = hi; *(uint32_t*)(Gs + (Q + tb) * SQ + t) = lo;
          }
        }
      }
      group_barrier(1);
      if (live) {
        const uint32_t ag = smem_u32(Gs + (16 * rt + (lane & 15)) * SQ + 8 * (lane >> 4));
        const uint32_t ax = smem_u32(Xc + lane * SP + 8 * NT * half);      // 32 tokens of one 8-column tile per load
#pragma unroll
        for (int jj = 0; jj < 2; ++jj) {
          if (2 * jj > rt) break;
          uint32_t b[NT][4], hi[2][4], lo[2][4];
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            if (2 * jj + u > rt) break;
            ldmatrix_x4(hi[u], ag + 32 * (2 * jj + u));
            ldmatrix_x4(lo[u], ag + (Q * SQ) * 2 + 32 * (2 * jj + u));
          }
#pragma unroll
          for (int n = 0; n < NT; ++n) ldmatrix_x4_trans(b[n], ax + (32 * jj * SP) * 2 + 16 * n);
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            if (2 * jj + u > rt) break;
#pragma unroll
            for (int n = 0; n < NT; ++n) {
              mma_bf16(Y[n], hi[u], b[n][2 * u], b[n][2 * u + 1]);
              mma_bf16(Z[n], lo[u], b[n][2 * u], b[n][2 * u + 1]);
            }
          }
        }
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) Y[n][e] += Z[n][e];
        const size_t ld = (size_t)p.H * p.P;
        const int col = 8 * NT * half + q2;
        float* dst = p.out + (size_t)(row0 + c * Q) * ld + off_x + col;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          if (ta < valid) {
            const float2 x = unpack2(*(const uint32_t*)(Xc + ta * SP + col + 8 * n));
            *(float2*)(dst + ta * ld + 8 * n) = make_float2(fmaf(D, x.x, Y[n][0]), fmaf(D, x.y, Y[n][1]));
          }
          if (tb < valid) {
            const float2 x = unpack2(*(const uint32_t*)(Xc + tb * SP + col + 8 * n));
            *(float2*)(dst + tb * ld + 8 * n) = make_float2(fmaf(D, x.x, Y[n][2]), fmaf(D, x.y, Y[n][3]));
          }
        }
      }
    } else {
      {                                                    // the weighted x: four threads per token, PB / 4 columns each
        const int t = (tid - 256) >> 2, c0 = (tid & 3) * (PB / 4);
        const float w = sc[3 * Q + t];
#pragma unroll
        for (int i = 0; i < PB / 16; ++i) {
          const int at = t * SP + c0 + 4 * i;
          const uint2 v = *(const uint2*)(Xc + at);
          const float2 a = unpack2(v.x), b = unpack2(v.y);
          uint2 hi, lo;
          split2(a.x * w, a.y * w, hi.x, lo.x);
          split2(b.x * w, b.y * w, hi.y, lo.y);
          *(uint2*)(Ws + at) = hi;
          *(uint2*)(Ws + Q * SP + at) = lo;
        }
      }
      const float all = sc[Q + Q - 1];                     // exp(L_last): tokens past the end decay nothing
#pragma unroll
      for (int i = 0; i < UM; ++i)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[i][n][e] *= all;
      group_barrier(2);
      const uint32_t aw = smem_u32(Ws + (lane & 15) * SP + 8 * (lane >> 4));
      const uint32_t at = smem_u32(Bc + (((lane >> 4) << 3) + (lane & 7)) * SN + 8 * ((lane >> 3) & 1));
#pragma unroll
      for (int k = 0; k < Q / 16; ++k) {
        if (16 * k >= valid) break;
#pragma unroll
        for (int i = 0; i < UM; ++i) {
          if (!own[i]) break;
          uint32_t a[4], b[4];
          ldmatrix_x4_trans(a, at + (16 * k * SN) * 2 + 2 * ur[i]);
          ldmatrix_x4_trans(b, aw + (16 * k * SP) * 2 + 2 * uc[i]);
          mma_bf16(S[i][0], a, b[0], b[1]);
          mma_bf16(S[i][1], a, b[2], b[3]);
          ldmatrix_x4_trans(b, aw + ((Q + 16 * k) * SP) * 2 + 2 * uc[i]);
          mma_bf16(S[i][0], a, b[0], b[1]);
          mma_bf16(S[i][1], a, b[2], b[3]);
        }
      }
      if (more) leave_state(st ^ 1);
      load_chunk(c + ST - 1);                              // into the place of chunk c - 1
      cp_async_wait<ST - 2>();
    }
    __syncthreads();
  }
  if (sw >= 0) {
#pragma unroll
    for (int i = 0; i < UM; ++i) {
      if (!own[i]) break;
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) sp[state_at(i, n, e)] = S[i][n][e];
    }
  }
}

template <int PB, int UM, int ST>
int launch_chunk(const SsdChunkArgs& a, int n_seg, cudaStream_t stream) {
  const size_t smem = 2 * (ST * Q * (2 * (size_t)pad_units(a.N) + pad_units(PB)) + 2 * Q * pad_units(PB) + 4 * (size_t)a.N * pad_units(PB) +
                           2 * Q * pad_units(Q)) + sizeof(float) * 8 * Q;
  static size_t allowed = 48 * 1024;
  if (smem > allowed) {
    if (smem > 227 * 1024) return FZ_TOO_LARGE;
    cudaError_t e = cudaFuncSetAttribute(ssd_chunk_kernel<PB, UM, ST>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    allowed = smem;
  }
  fz_launch(ssd_chunk_kernel<PB, UM, ST>, dim3(n_seg, a.H, a.P / PB), dim3(SSD_THREADS), smem, stream, a);
  FZ_LAUNCH_CHECK();
  return FZ_OK;
}
}  // namespace

// Sizes taken: state and value sizes that are multiples of 16, states of up to 256; x, B and C rows 16-byte aligned.
FZ_API int fz_ssd_chunk_check(const void* xbc, int H, int G, int N, int P) {
  if (H <= 0 || H > 65535 || G <= 0 || H % G || N <= 0 || N > 256 || N % 16 || P <= 0 || P % 16) return FZ_BAD_SHAPE;
  return ((uintptr_t)xbc & 15) == 0 ? FZ_OK : FZ_BAD_ALIGNMENT;
}

FZ_API int fz_ssd_chunk(const void* xbc, int H, int G, int N, int P, const float* dt, int ldt, int off_dt, const float* dt_bias,
                        const float* a_log, const float* skip, float* state, int npad, const int* seg, int n_seg, int min_rows,
                        float* out, cudaStream_t stream) {
  if (n_seg <= 0) return FZ_OK;
  int st = fz_ssd_chunk_check(xbc, H, G, N, P);
  if (st != FZ_OK) return st;
  if (npad < N || ((uintptr_t)out & 7)) return FZ_BAD_SHAPE;
  const SsdChunkArgs a = {(const __nv_bfloat16*)xbc, H * P + 2 * G * N, H, G, N, P, dt, ldt, off_dt, dt_bias, a_log, skip, state, npad,
                          seg, min_rows, out};
  // units of 16 state rows x 16 columns: N / 16 * PB / 16, eight warps
  if (P % 32 == 0 && N <= 128) return N <= 64 ? launch_chunk<32, 1, 3>(a, n_seg, stream) : launch_chunk<32, 2, 3>(a, n_seg, stream);
  return N <= 128 ? launch_chunk<16, 1, 3>(a, n_seg, stream) : launch_chunk<16, 2, 2>(a, n_seg, stream);
}

#ifdef FZ_TIMELINE
FZ_TIMELINE_READER(ssd_chunk)
#endif
