// Pieces shared by the recurrent scans whose state is a matrix per head: which part of the state a thread owns, its loads
// and stores, reductions over the lanes that share a column, copies into the staging area.
#pragma once
#include "common.cuh"

namespace {
// The state of a head is a key_dim x value_dim matrix S. A thread owns DPT = 8 consecutive rows of DC = 4 neighbouring
// columns, as sixteen packed pairs: the recurrence runs on packed float32 x 2 instructions (each half rounds as the scalar
// instruction does), every key and query value read from shared memory serves four columns, and a head is spread over
// value_dim / 4 x R threads (the kernels are bound by the instructions they issue per token, not by memory). The R lanes that share the columns (R a power of two, R * 8 >= key_dim; lane = r * (32 / R)
// + group, so that neighbouring lanes read one address of shared memory) add their partial dot products with shuffles.
// State layout in memory: (slots, heads, value_dim, R * 8), so a thread's 8 values of a column are contiguous and a
// column's run is read in 32-byte pieces; rows beyond key_dim stay zero. A block covers (blockDim / R) * 4 columns of one
// head of one portion and walks the portion's tokens in chunks, staged in shared memory by all threads.
constexpr int DPT = 8;
constexpr int DC = 4;                       // value columns per thread: two packed pairs
constexpr int SCAN_MAX_THREADS = 512;
// While a chunk of tokens is computed, the inputs of the next one travel from global into a raw staging area of shared
// memory (`cp.async`, four bytes each); after the chunk they are turned into what the recurrence reads (rotated or unit
// vectors, decays, gates) in a second area. tch: tokens per chunk (16, or 8 where shared memory would not hold 16).

// Sum over the R lanes that hold the rows of one column group: they are 32 / R lanes apart.
template <int R>
__device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
  for (int o = 16; o >= 32 / R; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Which column group (of the block) and which 16 rows a thread owns.
template <int R>
__device__ __forceinline__ void scan_place(int& group, int& r) {
  constexpr int per_warp = 32 / R;
  const int lane = threadIdx.x & 31;
  r = lane / per_warp;
  group = (threadIdx.x >> 5) * per_warp + lane % per_warp;
}

// The thread's 8 rows of two neighbouring columns (dkp floats apart), as pairs (column, column + 1); the second column
// is read and written only where it exists.
__device__ __forceinline__ void load_state(const float* __restrict__ p, int dkp, bool first, bool second, float2* S) {
#pragma unroll
  for (int i = 0; i < DPT; i += 4) {
    const float4 a = first ? *(const float4*)(p + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 b = second ? *(const float4*)(p + dkp + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    S[i] = make_float2(a.x, b.x); S[i + 1] = make_float2(a.y, b.y); S[i + 2] = make_float2(a.z, b.z); S[i + 3] = make_float2(a.w, b.w);
  }
}
__device__ __forceinline__ void store_state(float* __restrict__ p, int dkp, bool first, bool second, const float2* S) {
#pragma unroll
  for (int i = 0; i < DPT; i += 4) {
    if (first) *(float4*)(p + i) = make_float4(S[i].x, S[i + 1].x, S[i + 2].x, S[i + 3].x);
    if (second) *(float4*)(p + dkp + i) = make_float4(S[i].y, S[i + 1].y, S[i + 2].y, S[i + 3].y);
  }
}
__device__ __forceinline__ void load8(const float* p, float* v) {       // 8 floats from shared memory, 32-byte aligned
  const float4 a = *(const float4*)p, b = *(const float4*)(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ float2 both(float v) { return make_float2(v, v); }

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }
__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
  const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}
// Unit i of `vec` four-byte words (1 or 4) from src to dst.
__device__ __forceinline__ void cp_words(float* dst, const float* src, int i, int vec) {
  if (vec == 4) cp_async16(dst + 4 * i, src + 4 * i);
  else cp_async4(dst + i, src + i);
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// Unit i of a run of values of T from global to shared: a four-byte copy in flight (T is float, or a pair of 16-bit
// values where `words` says that source, destination and length allow it), else one value copied at once.
template <typename T>
__device__ __forceinline__ void stage_unit(T* dst, const T* src, int i, bool words) {
  if (sizeof(T) == 4) cp_async4(dst + i, src + i);
  else if (words) cp_async4(dst + 2 * i, src + 2 * i);
  else dst[i] = src[i];
}

int lanes_per_column(int dk) {
  int R = 1;
  while (R * DPT < dk) R <<= 1;
  return R;
}

template <typename K>
int allow_smem(K kern, size_t smem, size_t& allowed) {
  if (smem > allowed) {
    if (smem > 227 * 1024) return FZ_TOO_LARGE;
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    allowed = smem;
  }
  return FZ_OK;
}

// Threads of a scan block: R lanes for each group of DC of the head's value columns, a multiple of 32, SCAN_MAX_THREADS at most.
int scan_threads(int dv, int R) {
  const long long want = ((long long)((dv + DC - 1) / DC) * R + 31) / 32 * 32;
  return (int)(want < SCAN_MAX_THREADS ? want : SCAN_MAX_THREADS);
}
}  // namespace

#define FZ_BY_LANES(R, CALL)          \
  switch (R) {                        \
    case 1: return CALL(1);           \
    case 2: return CALL(2);           \
    case 4: return CALL(4);           \
    case 8: return CALL(8);           \
    case 16: return CALL(16);         \
    default: return CALL(32);         \
  }
