// Attention operands without rotation on packed batches: queries scaled by a factor of their position, values mixed with another
// layer's values of the same token, and means of blocks of cache rows.
//
// mixed_kv: a projection row holds q (H heads of dk), k (G of dk) and v (G of dv) at given columns; q is multiplied by
// q_factor[position], v becomes (1 - lambda) v + lambda v_first. The cache row [K of every kv head | V of every kv head] is written, q
// goes to [n_tok, H, dkp], and for whole prompts k and v also to dense operands of dkp, dvp features a head; features past dk / dv are
// zero there, so that a tensor-core kernel of the next larger width takes heads of any size.
//
// pool_rows: the mean of every whole block of P cache rows, taken of the rows as the cache holds them. With one token per sequence
// mixed_kv makes the mean itself, in the block that wrote the last row of a block of tokens.
//
// Factors, mixing and means are fp32. This file is built without fast-math.
#include "serve_common.cuh"
#include "serve_kernels.cuh"

namespace b200 {

namespace {

// V features from p on (V = 1 or a 16-byte vector)
template <typename T, int V>
__device__ __forceinline__ void load_n(const T* p, float (&f)[V]) {
  if constexpr (V == 1) f[0] = ldf(p);
  else Vec16<T>::load(p, f);
}
template <typename T, int V>
__device__ __forceinline__ void store_n(T* p, const float (&f)[V]) {
  if constexpr (V == 1)
    stf(p, f[0]);
  else if constexpr (sizeof(T) == 2)
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
  else
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}

// Mean of block `blk` over the features that this thread owns, handed to put(first feature, values).
template <typename T, int V, typename F>
__device__ __forceinline__ void block_mean(const PagedRows& pages, int P, int slot, int blk, F put) {
  const float inv = 1.f / P;
  const int first = blk * P, last = first + P - 1;
  const bool one_page = first / pages.page_size == last / pages.page_size;   // then its rows follow one another
  const int64_t row0 = page_row(pages, slot, first);
  for (int i = threadIdx.x * V; i < pages.width; i += blockDim.x * V) {
    float s[V];
#pragma unroll
    for (int j = 0; j < V; ++j) s[j] = 0.f;
#pragma unroll 8
    for (int r = 0; r < P; ++r) {
      const int64_t row = one_page ? row0 + r : page_row(pages, slot, first + r);
      float f[V];
      load_n<T, V>(static_cast<const T*>(pages.pool) + (row < 0 ? 0 : row) * pages.width + i, f);
#pragma unroll
      for (int j = 0; j < V; ++j) s[j] += f[j];
    }
#pragma unroll
    for (int j = 0; j < V; ++j) s[j] *= inv;
    put(i, s);
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256)
mixed_kv_kernel(const SeqBatch sb, const MixedKv a, const PagedRows pages, T* __restrict__ qo, T* __restrict__ ko, T* __restrict__ vo,
                bool single, int* status) {
  const int n = blockIdx.x, b = sb.tok_seq[n], off = n - sb.cu[b], pos = sb.start[b] + off, slot = sb.ids[b];
  const int64_t dst = page_row(pages, slot, pos);
  if (dst < 0 || (a.q_factor != nullptr && pos >= a.n_pos)) {
    if (threadIdx.x == 0) report_status(status, kBadArgument, 345, b, pos);
    return;
  }
  const T* row = static_cast<const T*>(a.in.y) + static_cast<int64_t>(n) * a.in.ld;
  const T* first = a.v_first != nullptr ? static_cast<const T*>(a.v_first) + static_cast<int64_t>(n) * a.ld_first : nullptr;
  T* cache = static_cast<T*>(pages.pool) + dst * pages.width;
  const float qf = a.q_factor != nullptr ? a.q_factor[pos] : 1.f, keep = 1.f - a.lambda;
  const int64_t dense = a.row0 != nullptr ? a.row0[b] + off : n;
  const int nq = a.H * a.dkp, nk = a.G * a.dkp, total = nq + nk + a.G * a.dvp;
  for (int i = threadIdx.x * V; i < total; i += blockDim.x * V) {
    float f[V];
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] = 0.f;
    if (i < nq) {
      const int h = i / a.dkp, c = i % a.dkp;
      if (c < a.dk) load_n<T, V>(row + a.in.q + h * a.dk + c, f);
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] *= qf;
      store_n<T, V>(qo + static_cast<int64_t>(n) * nq + i, f);
    } else if (i < nq + nk) {
      const int h = (i - nq) / a.dkp, c = (i - nq) % a.dkp;
      if (c < a.dk) {
        load_n<T, V>(row + a.in.k + h * a.dk + c, f);
        store_n<T, V>(cache + h * a.dk + c, f);
      }
      if (ko != nullptr) store_n<T, V>(ko + dense * nk + i - nq, f);
    } else {
      const int h = (i - nq - nk) / a.dvp, c = (i - nq - nk) % a.dvp;
      if (c < a.dv) {
        load_n<T, V>(row + a.in.v + h * a.dv + c, f);
        if (first != nullptr) {
          float g[V];
          load_n<T, V>(first + h * a.dv + c, g);
#pragma unroll
          for (int j = 0; j < V; ++j) f[j] = keep * f[j] + a.lambda * g[j];
        }
        store_n<T, V>(cache + a.G * a.dk + h * a.dv + c, f);
      }
      if (vo != nullptr) store_n<T, V>(vo + dense * (a.G * a.dvp) + i - nq - nk, f);
    }
  }
  if (!single || a.pooled == nullptr || (pos + 1) % a.pool != 0) return;
  __syncthreads();                         // the new row is part of the mean
  const int blk = pos / a.pool;
  T* out = static_cast<T*>(a.pooled) + pooled_row(pages, a.pool, slot, blk) * pages.width;
  block_mean<T, V>(pages, a.pool, slot, blk, [&](int i, const float (&s)[V]) { store_n<T, V>(out + i, s); });
}

template <typename T, int V>
__global__ void __launch_bounds__(128)
pool_rows_kernel(const SeqBatch sb, const MixedKv a, const PagedRows pages, const int* __restrict__ pad, T* __restrict__ ko, T* __restrict__ vo,
                 int* status) {
  const int P = a.pool;
  int unit = blockIdx.x, b = 0, blk = -1, whole = 0, dense_rows = 0;   // unit -> (sequence, block)
  for (; b < sb.n_seq; ++b) {
    const int s = sb.start[b], e = s + sb.cu[b + 1] - sb.cu[b], b0 = s / P;
    whole = e / P;
    dense_rows = pad != nullptr ? pad[b] : 0;
    const int units = max(whole, dense_rows) - b0;
    if (unit < units) {
      blk = b0 + unit;
      break;
    }
    unit -= max(units, 0);
  }
  if (blk < 0) return;
  const int wk = a.G * a.dkp, wv = a.G * a.dvp;
  T *kd = nullptr, *vd = nullptr;
  if (blk < dense_rows) {
    const int64_t r = a.row0[b] - dense_rows + blk;
    kd = ko + r * wk;
    vd = vo + r * wv;
    if (blk >= whole || a.dkp != a.dk || a.dvp != a.dv) {      // zeros, or zeros around the heads
      const float zero[V] = {};
      for (int i = threadIdx.x * V; i < wk; i += blockDim.x * V)
        if (blk >= whole || i % a.dkp >= a.dk) store_n<T, V>(kd + i, zero);
      for (int i = threadIdx.x * V; i < wv; i += blockDim.x * V)
        if (blk >= whole || i % a.dvp >= a.dv) store_n<T, V>(vd + i, zero);
    }
  }
  if (blk >= whole) return;
  const int64_t dst = pooled_row(pages, P, sb.ids[b], blk);
  if (dst < 0) {
    if (threadIdx.x == 0) report_status(status, kBadArgument, 346, b, blk);
    return;
  }
  T* out = static_cast<T*>(a.pooled) + dst * pages.width;
  const int nk = a.G * a.dk;
  block_mean<T, V>(pages, P, sb.ids[b], blk, [&](int i, const float (&s)[V]) {
    store_n<T, V>(out + i, s);
    if (kd == nullptr) return;
    if (i < nk) store_n<T, V>(kd + i / a.dk * a.dkp + i % a.dk, s);
    else store_n<T, V>(vd + (i - nk) / a.dv * a.dvp + (i - nk) % a.dv, s);
  });
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

bool fits_vectors(const MixedKv& a, int V) {
  const int64_t all = a.dk | a.dv | a.dkp | a.dvp | a.in.q | a.in.k | a.in.v | a.in.ld | (a.v_first != nullptr ? a.ld_first : 0);
  return all % V == 0 && aligned16(a.in.y) && aligned16(a.v_first);
}

bool bad_shape(const MixedKv& a, const PagedRows& pages) {
  return a.H < 1 || a.G < 1 || pages.width != a.G * (a.dk + a.dv) || a.dkp < a.dk || a.dvp < a.dv || (a.pooled != nullptr && a.pool < 1);
}

int threads_of(int units) { return units <= 64 ? 64 : units <= 128 ? 128 : 256; }

}  // namespace

cudaError_t launch_mixed_kv(bool f32, const SeqBatch& sb, const MixedKv& a, const PagedRows& pages, void* q, void* k, void* v, int* status,
                            cudaStream_t st) {
  if (bad_shape(a, pages)) return cudaErrorInvalidValue;
  const int V = f32 ? 4 : 8, features = (a.H + a.G) * a.dkp + a.G * a.dvp;
  const bool vec = fits_vectors(a, V), single = sb.n_tok == sb.n_seq;
  const int th = threads_of(vec ? features / V : features);
#define B200_MIX(T, N) mixed_kv_kernel<T, N><<<sb.n_tok, th, 0, st>>>(sb, a, pages, static_cast<T*>(q), static_cast<T*>(k), static_cast<T*>(v), single, status)
  if (f32) { if (vec) B200_MIX(float, 4); else B200_MIX(float, 1); }
  else { if (vec) B200_MIX(__nv_bfloat16, 8); else B200_MIX(__nv_bfloat16, 1); }
#undef B200_MIX
  return cudaGetLastError();
}

cudaError_t launch_pool_rows(bool f32, const SeqBatch& sb, const MixedKv& a, const PagedRows& pages, const int* pad, int n_rows, void* k,
                             void* v, int* status, cudaStream_t st) {
  if (bad_shape(a, pages) || a.pooled == nullptr || (pad != nullptr && (a.row0 == nullptr || k == nullptr || v == nullptr))) return cudaErrorInvalidValue;
  if (n_rows < 1) return cudaSuccess;
  const int V = f32 ? 4 : 8;
  const bool vec = ((a.dk | a.dv | a.dkp | a.dvp) % V) == 0;
  const int units = vec ? pages.width / V : pages.width, th = units <= 64 ? 64 : 128;
#define B200_POOL(T, N) pool_rows_kernel<T, N><<<n_rows, th, 0, st>>>(sb, a, pages, pad, static_cast<T*>(k), static_cast<T*>(v), status)
  if (f32) { if (vec) B200_POOL(float, 4); else B200_POOL(float, 1); }
  else { if (vec) B200_POOL(__nv_bfloat16, 8); else B200_POOL(__nv_bfloat16, 1); }
#undef B200_POOL
  return cudaGetLastError();
}

}  // namespace b200
