// Small helpers of the serving kernels: typed loads and stores, block reductions, page lookup.
#pragma once
#include "common.cuh"
#include "serve_kernels.cuh"
#include "softcap.cuh"

namespace b200 {

template <typename T>
__device__ __forceinline__ float ldf(const T* p);
template <>
__device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <>
__device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T>
__device__ __forceinline__ void stf(T* p, float v);
template <>
__device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <>
__device__ __forceinline__ void stf<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
// value after a round trip through the activation dtype
template <typename T>
__device__ __forceinline__ float rnd(float v);
template <>
__device__ __forceinline__ float rnd<float>(float v) { return v; }
template <>
__device__ __forceinline__ float rnd<__nv_bfloat16>(float v) { return __bfloat162float(__float2bfloat16(v)); }

// 16-byte vector of the activation dtype as floats
template <typename T>
struct Vec16;
template <>
struct Vec16<float> {
  static constexpr int n = 4;
  static __device__ __forceinline__ void load(const float* p, float (&f)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  }
};
template <>
struct Vec16<__nv_bfloat16> {
  static constexpr int n = 8;
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&f)[8]) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y), c = unpack_bf16x2(v.z), d = unpack_bf16x2(v.w);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
  }
};

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Sum over the block (blockDim.x a multiple of 32, at most 1024); `red` holds 33 floats. Every thread gets the sum.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < nw ? red[lane] : 0.f;
    t = warp_sum(t);
    if (lane == 0) red[32] = t;
  }
  __syncthreads();
  return red[32];
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ float lg2_approx(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float sqrt_approx(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
constexpr float kLog2e = 1.4426950408889634f;
__device__ __forceinline__ float sigmoid_approx(float x) { return rcp_approx(1.f + ex2_approx(-kLog2e * x)); }

// D += A B, m16n8k16, bf16 operands, fp32 sums: A rows are g and g + 8 of lane 4 g + t, B and D columns g and 2 t, 2 t + 1.
__device__ __forceinline__ void mma_bf16_16816(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// Row of position `pos` of cache slot `slot` in a page pool, or -1.
__device__ __forceinline__ int64_t page_row(const PagedRows& pg, int slot, int pos) {
  const int pi = pos / pg.page_size;
  if (pi >= pg.max_pages) return -1;
  const int page = pg.block_table[static_cast<int64_t>(slot) * pg.max_pages + pi];
  if (page < 0 || page >= pg.n_pages) return -1;
  return static_cast<int64_t>(page) * pg.page_size + pos % pg.page_size;
}

// Row of the mean of positions b P .. b P + P - 1 in a pool of such rows: it lies in the page of its last token, whose rows
// [page, 0 .. ceil(page_size / P)) hold the blocks that end there in order. -1: no such page.
__device__ __forceinline__ int64_t pooled_row(const PagedRows& pg, int P, int slot, int b) {
  const int pi = (b * P + P - 1) / pg.page_size;
  if (pi >= pg.max_pages) return -1;
  const int page = pg.block_table[static_cast<int64_t>(slot) * pg.max_pages + pi];
  if (page < 0 || page >= pg.n_pages) return -1;
  return static_cast<int64_t>(page) * ((pg.page_size + P - 1) / P) + b - pi * pg.page_size / P;
}
// Blocks of P tokens that lie wholly before the window of a query at `pos`.
__device__ __forceinline__ int blocks_seen(int pos, int window, int P) { return max(0, pos - window + 1) / P; }

// Opts a kernel into `bytes` of dynamic shared memory once per new maximum.
template <typename K>
inline cudaError_t want_smem(K kernel, int bytes, int& have) {
  if (bytes <= 48 * 1024 || bytes <= have) return cudaSuccess;
  if (bytes > 227 * 1024) return cudaErrorInvalidValue;
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e == cudaSuccess) have = bytes;
  return e;
}

}  // namespace b200
