// The scan of the selective state space mixer, token by token: per head a matrix state M (state size x value size) with
// one decay per token, M = exp(-exp(A) d) M + (d B) x^T, y = M^T C + D x, d = softplus(dt + bias). Everything is 32-bit;
// T is the type of x, B and C as the convolution left them. Long portions in bfloat16 have a kernel of their own
// (ssd_chunk.cu).
//
// Portions: seg[s] = (first row, rows, first position, state slot); a block walks a portion's tokens in order from the
// state in the request's slot and leaves the state there. A value's bits depend on its own sequence only.
#include "common.cuh"
#include "scan.cuh"
#include <math.h>

namespace {
__device__ __forceinline__ float softplus32(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// Unit i of a run of values of T: `bytes` = 16 or 4 bytes in flight per unit, or (0) one value copied at once.
template <typename T>
__device__ __forceinline__ void stage_piece(T* dst, const T* src, int i, int bytes) {
  if (bytes == 16) cp_async16(dst + i * (16 / (int)sizeof(T)), src + i * (16 / (int)sizeof(T)));
  else if (bytes == 4) cp_async4(dst + i * (4 / (int)sizeof(T)), src + i * (4 / (int)sizeof(T)));
  else dst[i] = src[i];
}

// xbc rows of W values: [x (H dv) | B (G dk) | C (G dk)]. Portions of more than max_rows rows are left alone. grid
// (portions, heads, slices of the value columns).
template <typename T, int R>
__global__ void __launch_bounds__(SCAN_MAX_THREADS)
ssd_scan_kernel(const T* __restrict__ xbc, int W, int H, int G, int dk, int dv, int tch, int bytes,
                const float* __restrict__ dt, int ldt, int off_dt, const float* __restrict__ dt_bias,
                const float* __restrict__ a_log, const float* __restrict__ skip, float* __restrict__ state,
                const int* __restrict__ seg, int max_rows, float* __restrict__ out) {
  fz_grid_launch_dependents();
  const int s = blockIdx.x, h = blockIdx.y;
  const int row0 = seg[4 * s], cnt = seg[4 * s + 1], slot = seg[4 * s + 3];
  const float rate = expf(a_log[h]), bias = dt_bias[h], D = skip[h];
  fz_grid_wait();
  if (cnt <= 0 || cnt > max_rows || slot < 0) return;
  extern __shared__ __align__(16) float smem[];
  const int NT = blockDim.x;
  const int dkp = R * DPT, COLS = NT / R * DC;
  const int dke = (dk + 7) & ~7, cole = (COLS + 7) & ~7;      // raw rows of T start on 16-byte boundaries
  float* cs = smem;                    // [tch][dkp]   C
  float* bs = cs + tch * dkp;          // [tch][dkp]   d B
  float* xs = bs + tch * dkp;          // [tch][COLS]  x, this block's columns
  float* gs = xs + tch * COLS;         // [tch]        decays
  float* rd = gs + tch;                // [tch]        raw: step sizes before bias and softplus
  T* rb = (T*)(rd + tch);              // [tch][dke]   raw: B, C, x
  T* rc = rb + tch * dke;
  T* rx = rc + tch * dke;              // [tch][cole]
  int group, r;
  scan_place<R>(group, r);
  const int col0 = blockIdx.z * COLS, col = col0 + group * DC;      // this thread's first column
  const int ncols = min(COLS, dv - col0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = h / (H / G);
  float* sp = state + (((size_t)slot * H + h) * dv + col) * dkp + r * DPT;
  const bool has[DC] = {col < dv, col + 1 < dv, col + 2 < dv, col + 3 < dv};
  float2 S[DC / 2][DPT];
  load_state(sp, dkp, has[0], has[1], S[0]);
  load_state(sp + 2 * (size_t)dkp, dkp, has[2], has[3], S[1]);
  const int per = bytes ? bytes / (int)sizeof(T) : 1;      // values per copy
  const int uk = dk / per, uv = ncols / per;
  const int per_token = 2 * uk + uv + 1;
  auto issue = [&](int t0) {
    const int tc = min(tch, cnt - t0);
    for (int e = threadIdx.x; e < tc * per_token; e += NT) {
      const int tt = e / per_token;
      int i = e - tt * per_token;
      const size_t n = (size_t)(row0 + t0 + tt);
      const T* in = xbc + n * W;
      if (i < uk) { stage_piece(rb + tt * dke, in + (size_t)H * dv + (size_t)g * dk, i, bytes); continue; }
      i -= uk;
      if (i < uk) { stage_piece(rc + tt * dke, in + (size_t)H * dv + (size_t)(G + g) * dk, i, bytes); continue; }
      i -= uk;
      if (i < uv) stage_piece(rx + tt * cole, in + (size_t)h * dv + col0, i, bytes);
      else cp_async4(rd + tt, dt + n * ldt + off_dt + h);
    }
    cp_async_commit();
  };
  auto cook = [&](int t0) {
    const int tc = min(tch, cnt - t0);
    for (int tt = warp; tt < tc; tt += NT / 32) {      // a warp cooks a token
      const float d = softplus32(rd[tt] + bias);
      if (lane == 0) gs[tt] = expf(-rate * d);
      for (int i = lane; i < dkp; i += 32) {
        bs[tt * dkp + i] = i < dk ? __fmul_rn(d, Cvt<T>::to_f(rb[tt * dke + i])) : 0.f;
        cs[tt * dkp + i] = i < dk ? Cvt<T>::to_f(rc[tt * dke + i]) : 0.f;
      }
      for (int c = lane; c < COLS; c += 32) xs[tt * COLS + c] = c < ncols ? Cvt<T>::to_f(rx[tt * cole + c]) : 0.f;
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
      const float4 v4 = *(const float4*)(xs + tt * COLS + group * DC);
      const float2 v[DC / 2] = {make_float2(v4.x, v4.y), make_float2(v4.z, v4.w)};
      const float2 dec = both(gs[tt]);
      float kk[DPT], qq[DPT];
      load8(bs + tt * dkp + r * DPT, kk);
      load8(cs + tt * dkp + r * DPT, qq);
      float2 o[DC / 2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
#pragma unroll
      for (int i = 0; i < DPT; ++i) {
        const float2 k2 = both(kk[i]), q2 = both(qq[i]);
#pragma unroll
        for (int j = 0; j < DC / 2; ++j) {
          S[j][i] = __ffma2_rn(dec, S[j][i], __fmul2_rn(k2, v[j]));
          o[j] = __ffma2_rn(S[j][i], q2, o[j]);
        }
      }
      const float res[DC] = {lanes_sum<R>(o[0].x), lanes_sum<R>(o[0].y), lanes_sum<R>(o[1].x), lanes_sum<R>(o[1].y)};
      if (r == 0) {
        const float x[DC] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
        for (int j = 0; j < DC; ++j)
          if (has[j]) dst[j] = __fmaf_rn(D, x[j], res[j]);
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

size_t ssd_smem(int dk, int R, int cols, int tch, size_t elem) {
  const int dkp = R * DPT;
  return sizeof(float) * (size_t)tch * ((size_t)2 * dkp + cols + 2) + elem * (size_t)tch * (2 * ((dk + 7) & ~7) + ((cols + 7) & ~7)) + 16;
}

template <typename T, int R>
int launch_ssd(const void* xbc, int W, int H, int G, int dk, int dv, const float* dt, int ldt, int off_dt, const float* dt_bias,
               const float* a_log, const float* skip, float* state, const int* seg, int n_seg, int max_rows, int cap, float* out,
               cudaStream_t stream) {
  int threads = scan_threads(dv, R);
  if (threads > cap) threads = cap;      // long portions: a head's columns are spread over several blocks
  if (threads < R) threads = R;
  const int cols = threads / R * DC;
  int tch = 16;
  while (tch > 2 && ssd_smem(dk, R, cols, tch, sizeof(T)) > 48 * 1024) tch >>= 1;
  const size_t smem = ssd_smem(dk, R, cols, tch, sizeof(T));
  static size_t allowed = 48 * 1024;
  int st = allow_smem(ssd_scan_kernel<T, R>, smem, allowed);
  if (st != FZ_OK) return st;
  // the widest copies that every run's start and length allow (runs of B and C, of a block's columns)
  const int es = (int)sizeof(T);
  const int last = dv % cols;
  auto fits = [&](int b) {
    return (dk * es) % b == 0 && (W * es) % b == 0 && (dv * es) % b == 0 && ((long long)H * dv * es) % b == 0 && (cols * es) % b == 0 &&
           (last * es) % b == 0 && ((uintptr_t)xbc % b) == 0;
  };
  const int bytes = fits(16) ? 16 : fits(4) ? 4 : 0;
  fz_launch(ssd_scan_kernel<T, R>, dim3(n_seg, H, (dv + cols - 1) / cols), dim3(threads), smem, stream, (const T*)xbc, W, H, G,
            dk, dv, tch, bytes, dt, ldt, off_dt, dt_bias, a_log, skip, state, seg, max_rows, out);
  FZ_LAUNCH_CHECK();
  return FZ_OK;
}
}  // namespace

// Portions of more than max_rows rows are passed over. threads: the most threads a block may have (a multiple of 32, at
// most 512).
FZ_API int fz_ssd_scan(const void* xbc, int dtype, int H, int G, int dk, int dv, const float* dt, int ldt, int off_dt,
                       const float* dt_bias, const float* a_log, const float* skip, float* state, const int* seg, int n_seg,
                       int max_rows, int threads, float* out, cudaStream_t stream) {
  if (n_seg <= 0) return FZ_OK;
  if (H <= 0 || H > 65535 || G <= 0 || H % G || dk <= 0 || dk > 32 * DPT || dv <= 0 || threads < 32 || threads % 32 ||
      threads > SCAN_MAX_THREADS) return FZ_BAD_SHAPE;
  const int W = H * dv + 2 * G * dk;
#define FZ_CALL_F(R) launch_ssd<float, R>(xbc, W, H, G, dk, dv, dt, ldt, off_dt, dt_bias, a_log, skip, state, seg, n_seg, max_rows, threads, out, stream)
#define FZ_CALL_B(R) launch_ssd<__nv_bfloat16, R>(xbc, W, H, G, dk, dv, dt, ldt, off_dt, dt_bias, a_log, skip, state, seg, n_seg, max_rows, threads, out, stream)
  if (dtype == FZ_F32) { FZ_BY_LANES(lanes_per_column(dk), FZ_CALL_F) }
  if (dtype == FZ_BF16) { FZ_BY_LANES(lanes_per_column(dk), FZ_CALL_B) }
#undef FZ_CALL_F
#undef FZ_CALL_B
  return FZ_BAD_DTYPE;
}

#ifdef FZ_TIMELINE
FZ_TIMELINE_READER(ssd)
#endif
