// The scan of gated linear attention: linear attention whose state decays per head and key channel by a number each token
// computes, token by token (see scan.cuh for what a thread owns and how tokens are staged).
//
//   alpha = sigmoid(z)^inv_root = exp(-inv_root * softplus(-z)),   S <- diag(alpha) S + k v^T,   o = S^T (q * q_scale)
//
// All arithmetic is 32-bit. Nothing depends on which other portions share the step.
#include "common.cuh"
#include "scan.cuh"
#include <math.h>

namespace {
__device__ __forceinline__ float softplus32(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// proj rows (ld floats): [q heads | k heads | v heads | ...]; z rows: H dk decay inputs. grid (portions, heads, column blocks).
// max_rows: portions of more rows are left to the kernel of long portions.
template <int R>
__global__ void __launch_bounds__(SCAN_MAX_THREADS)
channel_decay_scan_kernel(const float* __restrict__ proj, int ld, int H, int dk, int dv, int tch, const float* __restrict__ z,
                          float inv_root, float q_scale, float* __restrict__ state, const int* __restrict__ seg, int max_rows,
                          float* __restrict__ out) {
  fz_grid_launch_dependents();
  const int s = blockIdx.x, h = blockIdx.y;
  const int row0 = seg[4 * s], cnt = seg[4 * s + 1], slot = seg[4 * s + 3];
  fz_grid_wait();
  if (cnt <= 0 || cnt > max_rows || slot < 0) return;
  extern __shared__ __align__(16) float smem[];
  const int NT = blockDim.x;
  const int dkp = R * DPT, COLS = NT / R * DC;
  float* qs = smem;                    // [tch][dkp]   what the recurrence reads
  float* ks = qs + tch * dkp;
  float* as = ks + tch * dkp;          //              the decays
  float* vs = as + tch * dkp;          // [tch][COLS]
  float* rq = vs + tch * COLS;         // [tch][dk]    raw: as the projections left them
  float* rk = rq + tch * dk;
  float* rz = rk + tch * dk;
  float* rv = rz + tch * dk;           // [tch][COLS]
  int group, r;
  scan_place<R>(group, r);
  const int col0 = blockIdx.z * COLS, col = col0 + group * DC;      // this thread's first column
  const int ncols = min(COLS, dv - col0);
  float* sp = state + (((size_t)slot * H + h) * dv + col) * dkp + r * DPT;
  const bool has[DC] = {col < dv, col + 1 < dv, col + 2 < dv, col + 3 < dv};
  float2 S[DC / 2][DPT];
  load_state(sp, dkp, has[0], has[1], S[0]);
  load_state(sp + 2 * (size_t)dkp, dkp, has[2], has[3], S[1]);
  // copies of 16 bytes where every run starts on a 16-byte boundary and has a length that is a multiple of four
  const int vec = ((dk | ld | dv | ncols | (H * dk)) & 3) == 0 && aligned16(proj) && aligned16(z) ? 4 : 1;
  const int uq = dk / vec, uv = ncols / vec;
  const int per_token = 3 * uq + uv;
  auto issue = [&](int t0) {
    const int tc = min(tch, cnt - t0);
    for (int e = threadIdx.x; e < tc * per_token; e += NT) {
      const int tt = e / per_token;
      int i = e - tt * per_token;
      const size_t n = (size_t)(row0 + t0 + tt);
      const float* in = proj + n * ld;
      if (i < uq) { cp_words(rq + tt * dk, in + (size_t)h * dk, i, vec); continue; }
      i -= uq;
      if (i < uq) { cp_words(rk + tt * dk, in + (size_t)(H + h) * dk, i, vec); continue; }
      i -= uq;
      if (i < uq) { cp_words(rz + tt * dk, z + n * H * dk + (size_t)h * dk, i, vec); continue; }
      i -= uq;
      cp_words(rv + tt * COLS, in + (size_t)2 * H * dk + (size_t)h * dv + col0, i, vec);
    }
    cp_async_commit();
  };
  auto cook = [&](int t0) {
    const int tc = min(tch, cnt - t0);
    for (int e = threadIdx.x; e < tc * dkp; e += NT) {
      const int tt = e / dkp, i = e - tt * dkp;
      float qv = 0.f, kv = 0.f, av = 0.f;
      if (i < dk) {
        qv = __fmul_rn(rq[tt * dk + i], q_scale);
        kv = rk[tt * dk + i];
        av = expf(-inv_root * softplus32(-rz[tt * dk + i]));
      }
      qs[e] = qv;
      ks[e] = kv;
      as[e] = av;
    }
    for (int e = threadIdx.x; e < tc * COLS; e += NT) {
      const int c = e % COLS;
      vs[e] = c < ncols ? rv[e] : 0.f;
    }
  };

  issue(0);
  cp_async_wait();
  __syncthreads();
  cook(0);
  __syncthreads();
  for (int t0 = 0; t0 < cnt; t0 += tch) {
    const int tc = min(tch, cnt - t0);
    const bool more = t0 + tch < cnt;
    if (more) issue(t0 + tch);
    float* dst = out + (size_t)(row0 + t0) * H * dv + (size_t)h * dv + col;
#pragma unroll 2
    for (int tt = 0; tt < tc; ++tt, dst += (size_t)H * dv) {
      const float4 v4 = *(const float4*)(vs + tt * COLS + group * DC);
      const float2 v[DC / 2] = {make_float2(v4.x, v4.y), make_float2(v4.z, v4.w)};
      float kk[DPT], qq[DPT], aa[DPT];
      load8(ks + tt * dkp + r * DPT, kk);
      load8(as + tt * dkp + r * DPT, aa);
      load8(qs + tt * dkp + r * DPT, qq);
      float2 o[DC / 2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
#pragma unroll
      for (int i = 0; i < DPT; ++i) {
        const float2 k2 = both(kk[i]), q2 = both(qq[i]), a2 = both(aa[i]);
#pragma unroll
        for (int j = 0; j < DC / 2; ++j) {
          S[j][i] = __ffma2_rn(a2, S[j][i], __fmul2_rn(k2, v[j]));
          o[j] = __ffma2_rn(S[j][i], q2, o[j]);
        }
      }
      const float res[DC] = {lanes_sum<R>(o[0].x), lanes_sum<R>(o[0].y), lanes_sum<R>(o[1].x), lanes_sum<R>(o[1].y)};
      if (r == 0) {
#pragma unroll
        for (int j = 0; j < DC; ++j)
          if (has[j]) dst[j] = res[j];
      }
    }
    if (more) {
      cp_async_wait();
      __syncthreads();               // the next chunk's raw inputs have arrived; every thread is done with this chunk
      cook(t0 + tch);
      __syncthreads();
    }
  }
  store_state(sp, dkp, has[0], has[1], S[0]);
  store_state(sp + 2 * (size_t)dkp, dkp, has[2], has[3], S[1]);
}

size_t scan_smem(int dk, int R, int cols, int tch) {
  const int dkp = R * DPT;
  return sizeof(float) * (size_t)tch * ((size_t)3 * dkp + cols + 3 * dk + cols);
}

template <int R>
int launch_scan(const float* proj, int ld, int H, int dk, int dv, const float* z, float inv_root, float q_scale, float* state,
                const int* seg, int n_seg, int max_rows, float* out, cudaStream_t stream) {
  const int threads = scan_threads(dv, R), cols = threads / R * DC;
  const int tch = scan_smem(dk, R, cols, 16) <= 48 * 1024 ? 16 : 8;
  const size_t smem = scan_smem(dk, R, cols, tch);
  static size_t allowed = 48 * 1024;
  int st = allow_smem(channel_decay_scan_kernel<R>, smem, allowed);
  if (st != FZ_OK) return st;
  fz_launch(channel_decay_scan_kernel<R>, dim3(n_seg, H, (dv + cols - 1) / cols), dim3(threads), smem, stream, proj, ld, H, dk, dv,
            tch, z, inv_root, q_scale, state, seg, max_rows, out);
  FZ_LAUNCH_CHECK();
  return FZ_OK;
}
}  // namespace

FZ_API int fz_channel_decay_scan(const float* proj, int ld, int H, int dk, int dv, const float* z, float inv_root, float q_scale,
                                 float* state, const int* seg, int n_seg, int max_rows, float* out, cudaStream_t stream) {
  if (n_seg <= 0) return FZ_OK;
  if (H <= 0 || H > 65535 || dv <= 0 || dk <= 0 || dk > 32 * DPT || ld < H * (2 * dk + dv)) return FZ_BAD_SHAPE;
#define FZ_CALL(R) launch_scan<R>(proj, ld, H, dk, dv, z, inv_root, q_scale, state, seg, n_seg, max_rows, out, stream)
  FZ_BY_LANES(lanes_per_column(dk), FZ_CALL)
#undef FZ_CALL
}

#ifdef FZ_TIMELINE
FZ_TIMELINE_READER(gla)
#endif
