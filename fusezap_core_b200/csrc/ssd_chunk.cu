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
// A block owns PB value columns of one head of one portion. Warps 0 .. 3 compute the results of a chunk (16 tokens each),
// warps 4 .. 7 the state after it (rows 16 (warp - 4 + 4 i) of the state each) and leave it as operands for the next
// chunk's results; one barrier per chunk. The next chunk's rows travel by cp.async meanwhile.
#include "attn_mma.cuh"
#include <math.h>

namespace {
using namespace fzattn;
constexpr int Q = 64;                       // tokens per chunk
constexpr int SSD_THREADS = 256;
constexpr float LOG2E = 1.4426950408889634f;

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

// PB: value columns per block (16 or 32). MT: state rows / 64, rounded up (1, 2 or 4). grid (portions, heads, P / PB).
template <int PB, int MT>
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
  constexpr int SP = PB + 8;
  __nv_bfloat16* Cs = (__nv_bfloat16*)smem_raw;            // [2][Q][SN]
  __nv_bfloat16* Bs = Cs + 2 * Q * SN;                     // [2][Q][SN]
  __nv_bfloat16* Xs = Bs + 2 * Q * SN;                     // [2][Q][SP]
  __nv_bfloat16* Ms = Xs + 2 * Q * SP;                     // [2][2][N][SP]: the state before a chunk, rounding and rest
  float* scal = (float*)(Ms + 4 * N * SP);                 // [2][4][Q]: L in powers of two, exp(L), d, exp(L_last - L) d
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = lane >> 2, q2 = (lane & 3) * 2;           // an accumulator's row (and row + 8) and first column
  const int g = h / (p.H / p.G);
  const int nc = (cnt + Q - 1) / Q;
  const size_t off_x = (size_t)h * p.P + p0, off_b = (size_t)p.H * p.P + (size_t)g * N, off_c = off_b + (size_t)p.G * N;

  auto load_chunk = [&](int c) {
    const int st = c & 1, r = tid >> 2;                    // four threads per token
    const bool ok = c * Q + r < cnt;
    const __nv_bfloat16* in = p.xbc + (size_t)(row0 + (ok ? c * Q + r : 0)) * p.W;
    const uint32_t dc = smem_u32(Cs + (st * Q + r) * SN), db = smem_u32(Bs + (st * Q + r) * SN), dx = smem_u32(Xs + (st * Q + r) * SP);
    for (int j = tid & 3; j < 2 * KN; j += 4) {
      cp_async16(dc + 16 * j, in + off_c + 8 * j, ok);
      cp_async16(db + 16 * j, in + off_b + 8 * j, ok);
    }
    for (int j = tid & 3; j < PB / 8; j += 4) cp_async16(dx + 16 * j, in + off_x + 8 * j, ok);
    cp_async_commit();
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
    *(float2*)(sc + Q) = make_float2(exp2f(l0), exp2f(l1));
    *(float2*)(sc + 2 * Q) = make_float2(d0, d1);
    *(float2*)(sc + 3 * Q) = make_float2(exp2f(last - l0) * d0, exp2f(last - l1) * d1);
  };

  float S[MT][PB / 8][4];                                  // warps 4 .. 7: the state's rows 16 (warp - 4 + 4 i)
  auto leave_state = [&](int buf) {
    __nv_bfloat16* hi = Ms + (size_t)buf * 2 * N * SP;
    __nv_bfloat16* lo = hi + (size_t)N * SP;
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int mt = warp - 4 + 4 * i;
      if (mt >= KN) continue;
#pragma unroll
      for (int n = 0; n < PB / 8; ++n) {
        const int at = (16 * mt + gq) * SP + 8 * n + q2;
        uint32_t a, b;
        split2(S[i][n][0], S[i][n][1], a, b);
        *(uint32_t*)(hi + at) = a; *(uint32_t*)(lo + at) = b;
        split2(S[i][n][2], S[i][n][3], a, b);
        *(uint32_t*)(hi + at + 8 * SP) = a; *(uint32_t*)(lo + at + 8 * SP) = b;
      }
    }
  };
  float* sp = p.state + ((size_t)slot * p.H + h) * p.P * p.npad;

  load_chunk(0);
  if (warp >= 4) {
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int mt = warp - 4 + 4 * i;
#pragma unroll
      for (int n = 0; n < PB / 8; ++n) {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          S[i][n][e] = mt < KN ? sp[(size_t)(p0 + 8 * n + q2 + (e & 1)) * p.npad + 16 * mt + gq + (e & 2) * 4] : 0.f;
      }
    }
    leave_state(0);
    if (warp == 7) {
      float r0, r1;
      raw_steps(0, r0, r1);
      scalars(0, r0, r1);
    }
  }
  cp_async_wait<0>();
  __syncthreads();

  for (int c = 0; c < nc; ++c) {
    const int st = c & 1, valid = min(Q, cnt - c * Q);
    const bool more = c + 1 < nc;
    if (more) load_chunk(c + 1);
    const __nv_bfloat16* Cc = Cs + st * Q * SN;
    const __nv_bfloat16* Bc = Bs + st * Q * SN;
    const __nv_bfloat16* Xc = Xs + st * Q * SP;
    const float* sc = scal + st * 4 * Q;
    if (warp < 4) {
      if (16 * warp < valid) {
        float G[8][4], Y[PB / 8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) G[j][e] = 0.f;
#pragma unroll
        for (int n = 0; n < PB / 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) Y[n][e] = 0.f;
        const __nv_bfloat16* hi = Ms + (size_t)st * 2 * N * SP;
        const uint32_t ac = smem_u32(Cc + (16 * warp + (lane & 15)) * SN + 8 * (lane >> 4));
        const uint32_t ab = smem_u32(Bc + (((lane >> 4) << 3) + (lane & 7)) * SN + 8 * ((lane >> 3) & 1));
        const uint32_t am = smem_u32(hi + (lane & 15) * SP + 8 * (lane >> 4));
        const uint32_t rest = (uint32_t)(N * SP * 2);
#pragma unroll 2
        for (int k = 0; k < KN; ++k) {
          uint32_t a[4], b[4];
          ldmatrix_x4(a, ac + 32 * k);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            if (j > warp) break;                           // tokens after this warp's: not seen
            ldmatrix_x4(b, ab + (16 * j * SN) * 2 + 32 * k);
            mma_bf16(G[2 * j], a, b[0], b[1]);
            mma_bf16(G[2 * j + 1], a, b[2], b[3]);
          }
#pragma unroll
          for (int n = 0; n < PB / 16; ++n) {
            const uint32_t at = am + (16 * k * SP) * 2 + 32 * n;
            ldmatrix_x4_trans(b, at);
            mma_bf16(Y[2 * n], a, b[0], b[1]);
            mma_bf16(Y[2 * n + 1], a, b[2], b[3]);
            ldmatrix_x4_trans(b, at + rest);
            mma_bf16(Y[2 * n], a, b[0], b[1]);
            mma_bf16(Y[2 * n + 1], a, b[2], b[3]);
          }
        }
        const int ta = 16 * warp + gq, tb = ta + 8;        // this thread's two tokens
        const float la = sc[ta], lb = sc[tb], ea = sc[Q + ta], eb = sc[Q + tb];
#pragma unroll
        for (int n = 0; n < PB / 8; ++n) { Y[n][0] *= ea; Y[n][1] *= ea; Y[n][2] *= eb; Y[n][3] *= eb; }
        const uint32_t ax = smem_u32(Xc + (lane & 15) * SP + 8 * (lane >> 4));
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (j > warp) break;
          uint32_t hi4[4], lo4[4];
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const int t = 16 * j + 8 * u + q2;             // the earlier tokens of this thread's columns: t, t + 1
            const float2 l = *(const float2*)(sc + t), d = *(const float2*)(sc + 2 * Q + t);
            const float* w = G[2 * j + u];
            const float w0 = t <= ta ? w[0] * (exp2f(la - l.x) * d.x) : 0.f, w1 = t + 1 <= ta ? w[1] * (exp2f(la - l.y) * d.y) : 0.f;
            const float w2 = t <= tb ? w[2] * (exp2f(lb - l.x) * d.x) : 0.f, w3 = t + 1 <= tb ? w[3] * (exp2f(lb - l.y) * d.y) : 0.f;
            split2(w0, w1, hi4[2 * u], lo4[2 * u]);
            split2(w2, w3, hi4[2 * u + 1], lo4[2 * u + 1]);
          }
#pragma unroll
          for (int n = 0; n < PB / 16; ++n) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, ax + (16 * j * SP) * 2 + 32 * n);
            mma_bf16(Y[2 * n], hi4, b[0], b[1]);
            mma_bf16(Y[2 * n + 1], hi4, b[2], b[3]);
            mma_bf16(Y[2 * n], lo4, b[0], b[1]);
            mma_bf16(Y[2 * n + 1], lo4, b[2], b[3]);
          }
        }
        const size_t ld = (size_t)p.H * p.P;
        float* dst = p.out + (size_t)(row0 + c * Q) * ld + off_x + q2;
#pragma unroll
        for (int n = 0; n < PB / 8; ++n) {
          if (ta < valid) {
            const float2 x = unpack2(*(const uint32_t*)(Xc + ta * SP + 8 * n + q2));
            *(float2*)(dst + ta * ld + 8 * n) = make_float2(fmaf(D, x.x, Y[n][0]), fmaf(D, x.y, Y[n][1]));
          }
          if (tb < valid) {
            const float2 x = unpack2(*(const uint32_t*)(Xc + tb * SP + 8 * n + q2));
            *(float2*)(dst + tb * ld + 8 * n) = make_float2(fmaf(D, x.x, Y[n][2]), fmaf(D, x.y, Y[n][3]));
          }
        }
      }
    } else {
      float r0 = 0.f, r1 = 0.f;
      if (warp == 7 && more) raw_steps(c + 1, r0, r1);
      const float all = sc[Q + Q - 1];                     // exp(L_last): tokens past the end decay nothing
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int n = 0; n < PB / 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[i][n][e] *= all;
      const uint32_t ax = smem_u32(Xc + (lane & 15) * SP + 8 * (lane >> 4));
      const uint32_t at = smem_u32(Bc + (((lane >> 4) << 3) + (lane & 7)) * SN + 8 * ((lane >> 3) & 1));
#pragma unroll
      for (int k = 0; k < Q / 16; ++k) {
        if (16 * k >= valid) break;
        const float2 wa = *(const float2*)(sc + 3 * Q + 16 * k + q2), wb = *(const float2*)(sc + 3 * Q + 16 * k + 8 + q2);
        uint32_t xh[PB / 8][2], xl[PB / 8][2];
#pragma unroll
        for (int n = 0; n < PB / 16; ++n) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, ax + (16 * k * SP) * 2 + 32 * n);
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const float2 va = unpack2(b[2 * u]), vb = unpack2(b[2 * u + 1]);
            split2(va.x * wa.x, va.y * wa.y, xh[2 * n + u][0], xl[2 * n + u][0]);
            split2(vb.x * wb.x, vb.y * wb.y, xh[2 * n + u][1], xl[2 * n + u][1]);
          }
        }
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          const int mt = warp - 4 + 4 * i;
          if (mt >= KN) break;
          uint32_t a[4];
          ldmatrix_x4_trans(a, at + (16 * k * SN) * 2 + 32 * mt);
#pragma unroll
          for (int n = 0; n < PB / 8; ++n) {
            mma_bf16(S[i][n], a, xh[n][0], xh[n][1]);
            mma_bf16(S[i][n], a, xl[n][0], xl[n][1]);
          }
        }
      }
      if (more) {
        leave_state(st ^ 1);
        if (warp == 7) scalars(c + 1, r0, r1);
      }
    }
    cp_async_wait<0>();
    __syncthreads();
  }
  if (warp >= 4) {
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int mt = warp - 4 + 4 * i;
      if (mt >= KN) continue;
#pragma unroll
      for (int n = 0; n < PB / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          sp[(size_t)(p0 + 8 * n + q2 + (e & 1)) * p.npad + 16 * mt + gq + (e & 2) * 4] = S[i][n][e];
    }
  }
}

template <int PB, int MT>
int launch_chunk(const SsdChunkArgs& a, int n_seg, cudaStream_t stream) {
  const size_t smem = 2 * (4 * (size_t)Q * pad_units(a.N) + 2 * Q * (PB + 8) + 4 * (size_t)a.N * (PB + 8)) + sizeof(float) * 8 * Q;
  static size_t allowed = 48 * 1024;
  if (smem > allowed) {
    if (smem > 227 * 1024) return FZ_TOO_LARGE;
    cudaError_t e = cudaFuncSetAttribute(ssd_chunk_kernel<PB, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    allowed = smem;
  }
  fz_launch(ssd_chunk_kernel<PB, MT>, dim3(n_seg, a.H, a.P / PB), dim3(SSD_THREADS), smem, stream, a);
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
  if (P % 32 == 0 && N <= 128) {
    if (N <= 64) return launch_chunk<32, 1>(a, n_seg, stream);
    return launch_chunk<32, 2>(a, n_seg, stream);
  }
  if (N <= 64) return launch_chunk<16, 1>(a, n_seg, stream);
  if (N <= 128) return launch_chunk<16, 2>(a, n_seg, stream);
  return launch_chunk<16, 4>(a, n_seg, stream);
}

#ifdef FZ_TIMELINE
FZ_TIMELINE_READER(ssd_chunk)
#endif
