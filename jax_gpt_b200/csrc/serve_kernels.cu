// Serving kernels of models whose layers run on packed (ragged) batches with a 32-bit residual: sequence
// bookkeeping, embedding plus bigram table, norms (also post-norm + residual + next pre-norm in one pass), few-row linear
// layers (decode), multi-head latent attention over paged latent rows (RMS-normed latents, interleaved rotary part,
// absorbed weights, softmax with a sink), and experts chosen by a token table or by a sigmoid router.
//
// Every kernel exists for fp32 and bf16 activations; accumulation, norms, angles, scores and softmax are fp32 in both.
// This file is built without fast-math: the fp32 instances are meant to be exact to rounding.
#include "serve_kernels.cuh"

#include "serve_common.cuh"

namespace b200 {

namespace {

// ---- bookkeeping -------------------------------------------------------------------------------------------------
__global__ void seq_begin_kernel(const int* __restrict__ ids, const int* __restrict__ cu, const int* __restrict__ tokens,
                                 int n_seq, int max_slots, int* lens, int* prev, int* start, int* prev_tok, int* status) {
  const int b = blockIdx.x * blockDim.x + threadIdx.x;
  if (b >= n_seq) return;
  const int slot = ids[b], n = cu[b + 1] - cu[b];
  if (slot < 0 || slot >= max_slots || n < 1) {
    report_status(status, kBadArgument, 300, b, slot);
    start[b] = 0;
    prev_tok[b] = 0;
    return;
  }
  const int s = lens[slot];
  start[b] = s;
  lens[slot] = s + n;
  prev_tok[b] = prev[slot];
  prev[slot] = tokens[cu[b + 1] - 1];
}

template <typename T>
__global__ void embed_bigram_kernel(const SeqBatch sb, const int* __restrict__ tokens, const int* __restrict__ prev_tok,
                                    const T* __restrict__ embed, int vocab, const T* __restrict__ bigram, long long buckets,
                                    long long mul_prev, long long mul_cur, int D, float* __restrict__ x, int* status) {
  const int n = blockIdx.x;
  const int b = sb.tok_seq[n], first = sb.cu[b];
  const int tok = tokens[n];
  if (tok < 0 || tok >= vocab) {
    if (threadIdx.x == 0) report_status(status, kBadArgument, 301, n, tok);
    for (int i = threadIdx.x; i < D; i += blockDim.x) x[static_cast<int64_t>(n) * D + i] = 0.f;
    return;
  }
  const T* e = embed + static_cast<int64_t>(tok) * D;
  const T* g = nullptr;
  if (bigram != nullptr) {
    long long row = buckets;
    if (n > first || sb.start[b] > 0) {
      const long long p = n > first ? tokens[n - 1] : prev_tok[b];
      row = (p * mul_prev + tok * mul_cur) % buckets;
    }
    g = bigram + row * D;
  }
  for (int i = threadIdx.x; i < D; i += blockDim.x)
    x[static_cast<int64_t>(n) * D + i] = ldf(e + i) + (g != nullptr ? ldf(g + i) : 0.f);
}

// ---- norms -------------------------------------------------------------------------------------------------------
template <typename TO>
__global__ void norm_rows_kernel(int mode, const float* __restrict__ x, const float* __restrict__ gamma,
                                 const float* __restrict__ beta, TO* __restrict__ out, int D, float eps) {
  __shared__ float red[33];
  const float* xr = x + static_cast<int64_t>(blockIdx.x) * D;
  TO* o = out + static_cast<int64_t>(blockIdx.x) * D;
  float mu = 0.f;
  if (mode == 0) {
    float s = 0.f;
    for (int i = threadIdx.x; i < D; i += blockDim.x) s += xr[i];
    mu = block_sum(s, red) / D;
  }
  float v = 0.f;
  for (int i = threadIdx.x; i < D; i += blockDim.x) {
    const float d = xr[i] - mu;
    v += d * d;
  }
  const float inv = 1.f / sqrtf(block_sum(v, red) / D + eps);
  for (int i = threadIdx.x; i < D; i += blockDim.x) {
    float r = (xr[i] - mu) * inv * gamma[i];
    if (mode == 0 && beta != nullptr) r += beta[i];
    stf(o + i, r);
  }
}

// The same with the row in registers: D a multiple of 4, at most 1024 * kIt; a warp per row up to 1024, else a block.
template <typename TO, int kIt, int kThr>
__global__ void __launch_bounds__(256)
norm_rows_vec_kernel(int mode, const float* __restrict__ x, const float* __restrict__ gamma, const float* __restrict__ beta,
                     TO* __restrict__ out, int rows, int D, float eps) {
  __shared__ float red[33];
  constexpr int kPer = 256 / kThr;   // rows per block
  const int row = blockIdx.x * kPer + threadIdx.x / kThr, t = threadIdx.x % kThr;
  if (kThr == 32 && row >= rows) return;
  auto total = [&](float v) { return kThr == 32 ? warp_sum(v) : block_sum(v, red); };
  const float* xr = x + static_cast<int64_t>(row) * D;
  float4 v[kIt];
  float s = 0.f;
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + t) * 4;
    v[k] = i < D ? *reinterpret_cast<const float4*>(xr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    s += (v[k].x + v[k].y) + (v[k].z + v[k].w);
  }
  const float mu = mode == 0 ? total(s) / D : 0.f;
  float q = 0.f;
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    if ((k * kThr + t) * 4 < D) {
      v[k].x -= mu; v[k].y -= mu; v[k].z -= mu; v[k].w -= mu;
      q += (v[k].x * v[k].x + v[k].y * v[k].y) + (v[k].z * v[k].z + v[k].w * v[k].w);
    }
  }
  const float inv = 1.f / sqrtf(total(q) / D + eps);
  TO* o = out + static_cast<int64_t>(row) * D;
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + t) * 4;
    if (i < D) {
      const float4 g = *reinterpret_cast<const float4*>(gamma + i);
      float4 r = make_float4(v[k].x * inv * g.x, v[k].y * inv * g.y, v[k].z * inv * g.z, v[k].w * inv * g.w);
      if (mode == 0 && beta != nullptr) {
        const float4 b = *reinterpret_cast<const float4*>(beta + i);
        r.x += b.x; r.y += b.y; r.z += b.z; r.w += b.w;
      }
      if constexpr (sizeof(TO) == 2) *reinterpret_cast<uint2*>(o + i) = make_uint2(pack_bf16x2(r.x, r.y), pack_bf16x2(r.z, r.w));
      else *reinterpret_cast<float4*>(o + i) = r;
    }
  }
}

template <typename TO>
void norm_rows_go(int mode, const float* x, const float* gamma, const float* beta, TO* out, int rows, int D, float eps,
                  cudaStream_t st) {
  const bool vec = D % 4 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(gamma) |
                                   reinterpret_cast<uintptr_t>(beta) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  if (vec && D <= 512 && rows >= 64) norm_rows_vec_kernel<TO, 4, 32><<<(rows + 7) / 8, 256, 0, st>>>(mode, x, gamma, beta, out, rows, D, eps);
  else if (vec && D <= 1024) norm_rows_vec_kernel<TO, 1, 256><<<rows, 256, 0, st>>>(mode, x, gamma, beta, out, rows, D, eps);
  else if (vec && D <= 2048) norm_rows_vec_kernel<TO, 2, 256><<<rows, 256, 0, st>>>(mode, x, gamma, beta, out, rows, D, eps);
  else if (vec && D <= 4096) norm_rows_vec_kernel<TO, 4, 256><<<rows, 256, 0, st>>>(mode, x, gamma, beta, out, rows, D, eps);
  else if (vec && D <= 8192) norm_rows_vec_kernel<TO, 8, 256><<<rows, 256, 0, st>>>(mode, x, gamma, beta, out, rows, D, eps);
  else norm_rows_kernel<TO><<<rows, D >= 1024 ? 256 : (D >= 256 ? 128 : 64), 0, st>>>(mode, x, gamma, beta, out, D, eps);
}

// ---- post-norm into the residual, then the next pre-norm --------------------------------------------------------------
// x = (add ? x : 0) + rms(y) gpost, out = rms(x) gnext in one pass over the row (out null: the first half only).
template <typename TY, typename TO>
__global__ void residual_norm_kernel(const TY* __restrict__ y, const float* __restrict__ gpost, float* __restrict__ x, int add,
                                     const float* __restrict__ gnext, TO* __restrict__ out, int D, float eps) {
  __shared__ float red[33];
  const int64_t r0 = static_cast<int64_t>(blockIdx.x) * D;
  float s = 0.f;
  for (int i = threadIdx.x; i < D; i += blockDim.x) { const float v = ldf(y + r0 + i); s += v * v; }
  const float iy = 1.f / sqrtf(block_sum(s, red) / D + eps);
  s = 0.f;
  for (int i = threadIdx.x; i < D; i += blockDim.x) {
    const float v = (add ? x[r0 + i] : 0.f) + ldf(y + r0 + i) * iy * gpost[i];
    x[r0 + i] = v;
    s += v * v;
  }
  if (out == nullptr) return;
  const float ix = 1.f / sqrtf(block_sum(s, red) / D + eps);
  for (int i = threadIdx.x; i < D; i += blockDim.x) stf(out + r0 + i, x[r0 + i] * ix * gnext[i]);
}

template <typename T>
__device__ __forceinline__ float4 ld4(const T* p) {
  if constexpr (sizeof(T) == 2) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y);
    return make_float4(a.x, a.y, b.x, b.y);
  } else {
    return *reinterpret_cast<const float4*>(p);
  }
}

template <typename TY, typename TO, int kIt, int kThr>
__global__ void __launch_bounds__(256)
residual_norm_vec_kernel(const TY* __restrict__ y, const float* __restrict__ gpost, float* __restrict__ x, int add,
                         const float* __restrict__ gnext, TO* __restrict__ out, int rows, int D, float eps) {
  __shared__ float red[33];
  constexpr int kPer = 256 / kThr;   // rows per block
  const int row = blockIdx.x * kPer + threadIdx.x / kThr, t = threadIdx.x % kThr;
  if (kThr == 32 && row >= rows) return;
  auto total = [&](float v) { return kThr == 32 ? warp_sum(v) : block_sum(v, red); };
  const int64_t r0 = static_cast<int64_t>(row) * D;
  float4 v[kIt], a[kIt];
  float s = 0.f;
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + t) * 4;
    v[k] = a[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < D) {
      v[k] = ld4(y + r0 + i);
      if (add) a[k] = *reinterpret_cast<const float4*>(x + r0 + i);
    }
    s += (v[k].x * v[k].x + v[k].y * v[k].y) + (v[k].z * v[k].z + v[k].w * v[k].w);
  }
  const float iy = 1.f / sqrtf(total(s) / D + eps);
  s = 0.f;
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + t) * 4;
    if (i < D) {
      const float4 g = *reinterpret_cast<const float4*>(gpost + i);
      a[k].x += v[k].x * iy * g.x; a[k].y += v[k].y * iy * g.y; a[k].z += v[k].z * iy * g.z; a[k].w += v[k].w * iy * g.w;
      *reinterpret_cast<float4*>(x + r0 + i) = a[k];
      s += (a[k].x * a[k].x + a[k].y * a[k].y) + (a[k].z * a[k].z + a[k].w * a[k].w);
    }
  }
  if (out == nullptr) return;
  const float ix = 1.f / sqrtf(total(s) / D + eps);
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + t) * 4;
    if (i < D) {
      const float4 g = *reinterpret_cast<const float4*>(gnext + i);
      const float4 r = make_float4(a[k].x * ix * g.x, a[k].y * ix * g.y, a[k].z * ix * g.z, a[k].w * ix * g.w);
      if constexpr (sizeof(TO) == 2) *reinterpret_cast<uint2*>(out + r0 + i) = make_uint2(pack_bf16x2(r.x, r.y), pack_bf16x2(r.z, r.w));
      else *reinterpret_cast<float4*>(out + r0 + i) = r;
    }
  }
}

template <typename TY, typename TO>
void residual_norm_go(const TY* y, const float* gpost, float* x, int add, const float* gnext, TO* out, int rows, int D, float eps,
                      cudaStream_t st) {
  const bool vec = D % 4 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(gpost) |
                                   reinterpret_cast<uintptr_t>(gnext) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
#define B200_RN(IT, THR) \
  residual_norm_vec_kernel<TY, TO, IT, THR><<<THR == 32 ? (rows + 7) / 8 : rows, 256, 0, st>>>(y, gpost, x, add, gnext, out, rows, D, eps)
  if (vec && D <= 512 && rows >= 64) B200_RN(4, 32);
  else if (vec && D <= 1024) B200_RN(1, 256);
  else if (vec && D <= 2048) B200_RN(2, 256);
  else if (vec && D <= 4096) B200_RN(4, 256);
  else if (vec && D <= 8192) B200_RN(8, 256);
  else residual_norm_kernel<TY, TO><<<rows, D >= 1024 ? 256 : (D >= 256 ? 128 : 64), 0, st>>>(y, gpost, x, add, gnext, out, D, eps);
#undef B200_RN
}

// ---- few-row linear ------------------------------------------------------------------------------------------------
constexpr int kLinWarps = 8;

__device__ __forceinline__ float row_act(float v, const RowsOut& o) {
  if (o.act == kActRelu2) {
    const float r = fmaxf(v, 0.f);
    return r * r;
  }
  if (o.act == kActSilu) return silu_f(v);
  if (o.act == kActXielu) return (v > 0.f ? o.act_a * v * v : o.act_b * (expm1f(v) - v)) + 0.5f * v;
  return v;
}

template <typename T>
__device__ __forceinline__ void rows_store(const RowsOut& o, int m, int n, float v) {
  if (n >= o.n1) {
    o.y2[static_cast<int64_t>(m) * o.ldy2 + n - o.n1] = v;
    return;
  }
  v = row_act(v, o);
  const int64_t i = static_cast<int64_t>(m) * o.ldy + n;
  if (o.out_mode == 0) stf(static_cast<T*>(o.y) + i, v);
  else if (o.out_mode == 1) static_cast<float*>(o.y)[i] = v;
  else static_cast<float*>(o.y)[i] += v;
}

// A warp computes NR output features for up to MR rows; lanes stride the contraction in 16-byte vectors. kGlu (NR = 2):
// one feature silu(gate) * up, rows n and N + n of w.
template <typename T, int MR, int NR, bool kVec, bool kGlu>
__global__ void __launch_bounds__(kLinWarps * 32)
rows_linear_kernel(const T* __restrict__ x, int64_t ldx, const T* __restrict__ w, int64_t ldw, int M, int N, int K,
                   const RowsOut out) {
  static_assert(!kGlu || NR == 2, "gate and up");
  const int lane = threadIdx.x & 31;
  const int n0 = (blockIdx.x * kLinWarps + (threadIdx.x >> 5)) * (kGlu ? 1 : NR);
  const int m0 = blockIdx.y * MR;
  if (n0 >= N) return;
  float acc[MR][NR];
#pragma unroll
  for (int m = 0; m < MR; ++m)
#pragma unroll
    for (int r = 0; r < NR; ++r) acc[m][r] = 0.f;
  const T* wr[NR];
#pragma unroll
  for (int r = 0; r < NR; ++r) wr[r] = w + static_cast<int64_t>(kGlu ? n0 + r * N : (n0 + r < N ? n0 + r : n0)) * ldw;
  const T* xr[MR];
#pragma unroll
  for (int m = 0; m < MR; ++m) xr[m] = x + static_cast<int64_t>(m0 + m < M ? m0 + m : m0) * ldx;
  if constexpr (kVec) {
    constexpr int V = Vec16<T>::n;
#pragma unroll (MR == 1 ? 4 : 2)
    for (int k = lane * V; k < K; k += 32 * V) {
      float wv[NR][V];
#pragma unroll
      for (int r = 0; r < NR; ++r) Vec16<T>::load(wr[r] + k, wv[r]);
#pragma unroll
      for (int m = 0; m < MR; ++m) {
        float xv[V];
        Vec16<T>::load(xr[m] + k, xv);
#pragma unroll
        for (int r = 0; r < NR; ++r)
#pragma unroll
          for (int j = 0; j < V; ++j) acc[m][r] = fmaf(xv[j], wv[r][j], acc[m][r]);
      }
    }
  } else {
    for (int k = lane; k < K; k += 32) {
#pragma unroll
      for (int m = 0; m < MR; ++m) {
        const float xv = ldf(xr[m] + k);
#pragma unroll
        for (int r = 0; r < NR; ++r) acc[m][r] = fmaf(xv, ldf(wr[r] + k), acc[m][r]);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < MR; ++m)
#pragma unroll
    for (int r = 0; r < NR; ++r) acc[m][r] = warp_sum(acc[m][r]);
#pragma unroll
  for (int m = 0; m < MR; ++m) {
    if constexpr (kGlu) {
      if (lane == m && m0 + m < M) rows_store<T>(out, m0 + m, n0, silu_f(acc[m][0]) * acc[m][1]);
    } else {
#pragma unroll
      for (int r = 0; r < NR; ++r)
        if (lane == ((m * NR + r) & 31) && m0 + m < M && n0 + r < N) rows_store<T>(out, m0 + m, n0 + r, acc[m][r]);
    }
  }
}

template <typename T, int MR, int NR, bool kGlu>
void rows_linear_go(bool vec, const T* x, int64_t ldx, const T* w, int64_t ldw, int M, int N, int K, const RowsOut& out,
                    cudaStream_t st) {
  constexpr int kPer = kLinWarps * (kGlu ? 1 : NR);
  const dim3 grid((N + kPer - 1) / kPer, (M + MR - 1) / MR);
  if (vec) rows_linear_kernel<T, MR, NR, true, kGlu><<<grid, kLinWarps * 32, 0, st>>>(x, ldx, w, ldw, M, N, K, out);
  else rows_linear_kernel<T, MR, NR, false, kGlu><<<grid, kLinWarps * 32, 0, st>>>(x, ldx, w, ldw, M, N, K, out);
}

// bf16, up to 8 * MT rows: weights are the A operand of mma.sync m16n8k16 (16 output features), activation rows the B
// operand. Every lane loads 16 contiguous bytes of a weight row and of an activation row; the products' k index is
// permuted the same way on both sides, which leaves the sums unchanged. The warps of a block split the contraction.
// Bound by the stream of weights: tcgen05 tiles would be 94 % padding here.
template <int MT, int kW, bool kGlu>   // kW warps per block
__global__ void __launch_bounds__(kW * 32)
rows_linear_mma_kernel(const __nv_bfloat16* __restrict__ x, int64_t ldx, const __nv_bfloat16* __restrict__ w, int64_t ldw,
                       int M, int N, int K, const RowsOut out) {
  constexpr int kMat = kGlu ? 2 : 1;   // gate (and up) weights
  __shared__ float red[kMat][kW][MT][32][4];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int n0 = blockIdx.x * 16;
  const __nv_bfloat16* w0 = w + static_cast<int64_t>(min(n0 + g, N - 1)) * ldw;
  const __nv_bfloat16* w1 = w + static_cast<int64_t>(min(n0 + g + 8, N - 1)) * ldw;
  const int64_t up = static_cast<int64_t>(N) * ldw;
  const __nv_bfloat16* xr[MT];
#pragma unroll
  for (int m = 0; m < MT; ++m) xr[m] = x + static_cast<int64_t>(min(m * 8 + g, M - 1)) * ldx;
  float acc[kMat][MT][4];
#pragma unroll
  for (int q = 0; q < kMat; ++q)
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[q][m][j] = 0.f;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  constexpr int kU = MT == 1 ? 4 : 2;
  for (int kb = warp * 32; kb < K; kb += kW * 32 * kU) {
    uint4 a[kMat][kU], c[kMat][kU], b[kU][MT];
#pragma unroll
    for (int u = 0; u < kU; ++u) {
      const int k = kb + u * kW * 32 + t * 8;
      const bool in = k < K;   // K is a multiple of 8
#pragma unroll
      for (int q = 0; q < kMat; ++q) {
        a[q][u] = in ? __ldg(reinterpret_cast<const uint4*>(w0 + q * up + k)) : zero;
        c[q][u] = in ? __ldg(reinterpret_cast<const uint4*>(w1 + q * up + k)) : zero;
      }
#pragma unroll
      for (int m = 0; m < MT; ++m) b[u][m] = in ? __ldg(reinterpret_cast<const uint4*>(xr[m] + k)) : zero;
    }
#pragma unroll
    for (int u = 0; u < kU; ++u)
#pragma unroll
      for (int q = 0; q < kMat; ++q)
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16_16816(acc[q][m], a[q][u].x, c[q][u].x, a[q][u].y, c[q][u].y, b[u][m].x, b[u][m].y);
          mma_bf16_16816(acc[q][m], a[q][u].z, c[q][u].z, a[q][u].w, c[q][u].w, b[u][m].z, b[u][m].w);
        }
  }
#pragma unroll
  for (int q = 0; q < kMat; ++q)
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < 4; ++j) red[q][warp][m][lane][j] = acc[q][m][j];
  __syncthreads();
  // accumulator j of lane (g, t): feature g + 8 * (j / 2), row 2 t + j % 2
  for (int i = threadIdx.x; i < MT * 128; i += kW * 32) {
    const int m = i / 128, f = i % 16, r = (i / 16) % 8;
    const int src = (f % 8) * 4 + r / 2, j = (f / 8) * 2 + r % 2;
    float v[kMat];
#pragma unroll
    for (int p = 0; p < kMat; ++p) {
      v[p] = 0.f;
#pragma unroll
      for (int q = 0; q < kW; ++q) v[p] += red[p][q][m][src][j];
    }
    if (m * 8 + r < M && n0 + f < N) rows_store<__nv_bfloat16>(out, m * 8 + r, n0 + f, kGlu ? silu_f(v[0]) * v[kMat - 1] : v[0]);
  }
}

template <int MT, bool kGlu>
void rows_linear_mma_go(const __nv_bfloat16* x, int64_t ldx, const __nv_bfloat16* w, int64_t ldw, int M, int N, int K,
                        const RowsOut& out, cudaStream_t st) {
  const int grid = (N + 15) / 16;   // wide outputs: small blocks, so that all of them are resident at once
  if (grid >= 296) rows_linear_mma_kernel<MT, 4, kGlu><<<grid, 128, 0, st>>>(x, ldx, w, ldw, M, N, K, out);
  else rows_linear_mma_kernel<MT, 8, kGlu><<<grid, 256, 0, st>>>(x, ldx, w, ldw, M, N, K, out);
}

template <typename T, bool kGlu>
cudaError_t rows_linear_t(const void* x, int64_t ldx, const void* w, int64_t ldw, int M, int N, int K, const RowsOut& out,
                          cudaStream_t st) {
  const bool vec = K % Vec16<T>::n == 0 && ldx % Vec16<T>::n == 0 && ldw % Vec16<T>::n == 0 &&
                   (reinterpret_cast<uintptr_t>(x) & 15) == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0;
  const T* xt = static_cast<const T*>(x);
  const T* wt = static_cast<const T*>(w);
  if constexpr (sizeof(T) == 2) {
    if (vec && M > 1 && M <= 32) {
      if (M <= 8) rows_linear_mma_go<1, kGlu>(xt, ldx, wt, ldw, M, N, K, out, st);
      else if (M <= 16) rows_linear_mma_go<2, kGlu>(xt, ldx, wt, ldw, M, N, K, out, st);
      else rows_linear_mma_go<4, kGlu>(xt, ldx, wt, ldw, M, N, K, out, st);
      return cudaGetLastError();
    }
  }
  // narrow outputs take fewer features per warp so that the grid still covers the SMs
#define B200_GO(MR)                                                                                       \
  {                                                                                                       \
    if constexpr (kGlu) rows_linear_go<T, MR, 2, true>(vec, xt, ldx, wt, ldw, M, N, K, out, st);          \
    else if (MR > 1 && N >= 148 * kLinWarps * 4) rows_linear_go<T, MR, 4, false>(vec, xt, ldx, wt, ldw, M, N, K, out, st); \
    else if (N >= 148 * kLinWarps * 2) rows_linear_go<T, MR, 2, false>(vec, xt, ldx, wt, ldw, M, N, K, out, st); \
    else rows_linear_go<T, MR, 1, false>(vec, xt, ldx, wt, ldw, M, N, K, out, st);                        \
  }
  if (M == 1) B200_GO(1)
  else if (M == 2) B200_GO(2)
  else if (M <= 4) B200_GO(4)
  else B200_GO(8)
#undef B200_GO
  return cudaGetLastError();
}

// ---- multi-head latent attention ------------------------------------------------------------------------------------
// Feature i of a rotary part read through `at(i)`, turned to position `pos`.
template <typename F>
__device__ __forceinline__ float rotated(const RopeTable& r, int pos, int i, F at) {
  if (i >= r.dims) return at(i);
  const int64_t k = static_cast<int64_t>(pos) * (r.dims / 2) + (i >> 1);
  const float c = r.cos[k], s = r.sin[k];
  return (i & 1) == 0 ? at(i) * c - at(i + 1) * s : at(i) * c + at(i - 1) * s;
}

// kHold > 0: the first kHold features of every thread stay in registers (turned where they turn), so that one wait covers all loads; for
// steps of a few tokens, where latency is all there is.
template <typename T, int kHold>
__global__ void mla_prepare_kernel(const SeqBatch sb, const T* __restrict__ y, int64_t ldy, int q_rank, int R, int dr,
                                   const float* __restrict__ q_gamma, const float* __restrict__ kv_gamma, float eps,
                                   const RopeTable rope, const PagedRows pages, T* __restrict__ cq, T* __restrict__ lat,
                                   int* status) {
  __shared__ float red[33];
  const int n = blockIdx.x;
  const int b = sb.tok_seq[n];
  const int pos = sb.start[b] + n - sb.cu[b];
  const T* row = y + static_cast<int64_t>(n) * ldy;
  const T* kv = row + q_rank;
  const int64_t dst = page_row(pages, sb.ids[b], pos);
  if (dst < 0 || pos >= rope.max_pos) {
    if (threadIdx.x == 0) report_status(status, kBadArgument, 302, b, pos);
    return;
  }
  auto turned = [&](int i) { return rotated(rope, pos, i - R, [&](int j) { return ldf(kv + R + j); }); };
  float held[kHold > 0 ? kHold : 1], gain[kHold > 0 ? kHold : 1];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int k = 0; k < kHold; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    held[k] = i < R ? ldf(kv + i) : (i < R + dr ? turned(i) : 0.f);
    gain[k] = i < R ? kv_gamma[i] : 0.f;
    if (i < R) sk += held[k] * held[k];
  }
  for (int i = threadIdx.x + kHold * blockDim.x; i < R; i += blockDim.x) { const float v = ldf(kv + i); sk += v * v; }
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) { const float v = ldf(row + i); sq += v * v; }
  const float iq = q_rank > 0 ? 1.f / sqrtf(block_sum(sq, red) / q_rank + eps) : 0.f;
  const float ik = 1.f / sqrtf(block_sum(sk, red) / R + eps);
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x)
    stf(cq + static_cast<int64_t>(n) * q_rank + i, ldf(row + i) * iq * q_gamma[i]);
  T* prow = static_cast<T*>(pages.pool) + dst * pages.width;
  T* lrow = lat != nullptr ? lat + static_cast<int64_t>(n) * (R + dr) : nullptr;
  auto put = [&](int i, float v) {
    stf(prow + i, v);
    if (lrow != nullptr) stf(lrow + i, v);
  };
#pragma unroll
  for (int k = 0; k < kHold; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < R + dr) put(i, i < R ? held[k] * ik * gain[k] : held[k]);
  }
  for (int i = threadIdx.x + kHold * blockDim.x; i < R + dr; i += blockDim.x) put(i, i < R ? ldf(kv + i) * ik * kv_gamma[i] : turned(i));
}

// One block per token: query heads rotated in place, keys assembled.
template <typename T>
__global__ void mla_rope_qk_kernel(const SeqBatch sb, T* __restrict__ q, int64_t ldq, const T* __restrict__ kn, int64_t ldkn,
                                   const T* __restrict__ lat, int64_t ldlat, int R, T* __restrict__ k, int H, int dn, int dr,
                                   const RopeTable rope) {
  const int n = blockIdx.x;
  const int b = sb.tok_seq[n];
  const int pos = sb.start[b] + n - sb.cu[b];
  const int half = rope.dims / 2, D = dn + dr;
  T* qr = q + static_cast<int64_t>(n) * ldq;
  for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
    const int h = i / half, j = i % half;
    const float c = rope.cos[static_cast<int64_t>(pos) * half + j], s = rope.sin[static_cast<int64_t>(pos) * half + j];
    T* p = qr + h * D + dn + 2 * j;
    const float u = ldf(p), v = ldf(p + 1);
    stf(p, u * c - v * s);
    stf(p + 1, v * c + u * s);
  }
  const T* kr = kn + static_cast<int64_t>(n) * ldkn;
  const T* rr = lat + static_cast<int64_t>(n) * ldlat + R;
  T* ko = k + static_cast<int64_t>(n) * H * D;
  constexpr int V = Vec16<T>::n;
  if (dn % V == 0 && dr % V == 0 && ldkn % V == 0 && ldlat % V == 0 && R % V == 0) {
    for (int i = threadIdx.x; i < H * D / V; i += blockDim.x) {
      const int h = i * V / D, j = i * V % D;
      const T* src = j < dn ? kr + h * dn + j : rr + (j - dn);
      *reinterpret_cast<uint4*>(ko + i * V) = *reinterpret_cast<const uint4*>(src);
    }
  } else {
    for (int i = threadIdx.x; i < H * D; i += blockDim.x) {
      const int h = i / D, j = i % D;
      ko[i] = j < dn ? kr[h * dn + j] : rr[j - dn];
    }
  }
}

constexpr int kAbsTok = 8;    // tokens per block of the absorption kernels
constexpr int kAbsCols = 64;  // latent columns per block of the query absorption

// Block: 8 tokens, one head, 64 columns. Lanes 0..7 of every eight own eight columns each, the other lane bits and
// the warps split the contraction over dn; partial sums meet in shuffles and in shared memory.
template <typename T, bool kVec>
__global__ void __launch_bounds__(256)
mla_absorb_q_kernel(const SeqBatch sb, const T* __restrict__ q, int64_t ldq, const T* __restrict__ w_uk, T* __restrict__ qf, int H, int dn,
                    int dr, int R, const RopeTable rope) {
  extern __shared__ float sm[];   // [kAbsTok][dn + dr], then [8 warps][kAbsTok][kAbsCols]
  const int D = dn + dr, h = blockIdx.y, n0 = blockIdx.x * kAbsTok;
  float* red = sm + kAbsTok * D;
  const int cnt = min(kAbsTok, sb.n_tok - n0);
  for (int i = threadIdx.x; i < kAbsTok * D; i += blockDim.x)
    sm[i] = i < cnt * D ? ldf(q + static_cast<int64_t>(n0 + i / D) * ldq + h * D + i % D) : 0.f;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c0 = blockIdx.z * kAbsCols + (lane & 7) * 8, dg = warp * 4 + (lane >> 3);   // 32 slices of dn
  const T* w = w_uk + static_cast<int64_t>(h) * dn * R;
  float acc[kAbsTok][8];
#pragma unroll
  for (int t = 0; t < kAbsTok; ++t)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[t][j] = 0.f;
#pragma unroll 2
  for (int d = dg; d < dn; d += 32) {
    float wv[8];
    if constexpr (kVec) {
      if (c0 < R) {
        if constexpr (sizeof(T) == 2) {
          Vec16<T>::load(w + static_cast<int64_t>(d) * R + c0, wv);
        } else {
          float f[4];
          Vec16<T>::load(w + static_cast<int64_t>(d) * R + c0, f);
          wv[0] = f[0]; wv[1] = f[1]; wv[2] = f[2]; wv[3] = f[3];
          Vec16<T>::load(w + static_cast<int64_t>(d) * R + c0 + 4, f);
          wv[4] = f[0]; wv[5] = f[1]; wv[6] = f[2]; wv[7] = f[3];
        }
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) wv[j] = 0.f;
      }
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) wv[j] = c0 + j < R ? ldf(w + static_cast<int64_t>(d) * R + c0 + j) : 0.f;
    }
#pragma unroll
    for (int t = 0; t < kAbsTok; ++t) {
      const float x = sm[t * D + d];
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[t][j] = fmaf(x, wv[j], acc[t][j]);
    }
  }
#pragma unroll
  for (int t = 0; t < kAbsTok; ++t)
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      float v = acc[t][j];
      v += __shfl_xor_sync(0xffffffffu, v, 8);
      v += __shfl_xor_sync(0xffffffffu, v, 16);
      if ((lane >> 3) == (t & 3)) red[(warp * kAbsTok + t) * kAbsCols + (lane & 7) * 8 + j] = v;
    }
  __syncthreads();
  for (int i = threadIdx.x; i < cnt * kAbsCols; i += blockDim.x) {
    const int t = i / kAbsCols, c = i % kAbsCols, r = blockIdx.z * kAbsCols + c;
    if (r < R) {
      float v = 0.f;
#pragma unroll
      for (int k = 0; k < 8; ++k) v += red[(k * kAbsTok + t) * kAbsCols + c];
      stf(qf + (static_cast<int64_t>(n0 + t) * H + h) * (R + dr) + r, v);
    }
  }
  if (blockIdx.z == 0)
    for (int i = threadIdx.x; i < cnt * dr; i += blockDim.x) {
      const int t = i / dr, j = i % dr, n = n0 + t, b = sb.tok_seq[n];
      const int pos = sb.start[b] + n - sb.cu[b];
      stf(qf + (static_cast<int64_t>(n) * H + h) * (R + dr) + R + j,
          rotated(rope, min(pos, rope.max_pos - 1), j, [&](int k) { return sm[t * D + dn + k]; }));
    }
}

// A warp computes one value feature of a head for up to 8 tokens; lanes stride the latent.
template <typename T, bool kVec>
__global__ void __launch_bounds__(256)
mla_absorb_out_kernel(const T* __restrict__ o_lat, const T* __restrict__ w_uv, const T* __restrict__ gate, int64_t ldg,
                      T* __restrict__ o, int n_tok, int H, int dv, int R) {
  extern __shared__ float sm[];   // [kAbsTok][R]
  const int h = blockIdx.y, n0 = blockIdx.x * kAbsTok;
  const int cnt = min(kAbsTok, n_tok - n0);
  if constexpr (kVec) {
    constexpr int V = Vec16<T>::n;
    for (int i = threadIdx.x * V; i < kAbsTok * R; i += blockDim.x * V) {
      float f[V];
      if (i < cnt * R) Vec16<T>::load(o_lat + (static_cast<int64_t>(n0 + i / R) * H + h) * R + i % R, f);
#pragma unroll
      for (int j = 0; j < V; ++j) sm[i + j] = i < cnt * R ? f[j] : 0.f;
    }
  } else {
    for (int i = threadIdx.x; i < kAbsTok * R; i += blockDim.x)
      sm[i] = i < cnt * R ? ldf(o_lat + (static_cast<int64_t>(n0 + i / R) * H + h) * R + i % R) : 0.f;
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  for (int v = blockIdx.z * nw + warp; v < dv; v += gridDim.z * nw) {
    const T* w = w_uv + (static_cast<int64_t>(h) * dv + v) * R;
    float acc[kAbsTok];
#pragma unroll
    for (int t = 0; t < kAbsTok; ++t) acc[t] = 0.f;
    if constexpr (kVec) {
      constexpr int V = Vec16<T>::n;
#pragma unroll 2
      for (int r = lane * V; r < R; r += 32 * V) {
        float wv[V];
        Vec16<T>::load(w + r, wv);
#pragma unroll
        for (int t = 0; t < kAbsTok; ++t)
#pragma unroll
          for (int j = 0; j < V; j += 4) {
            const float4 x = *reinterpret_cast<const float4*>(sm + t * R + r + j);
            acc[t] = fmaf(x.x, wv[j], fmaf(x.y, wv[j + 1], fmaf(x.z, wv[j + 2], fmaf(x.w, wv[j + 3], acc[t]))));
          }
      }
    } else {
#pragma unroll 4
      for (int r = lane; r < R; r += 32) {
        const float wv = ldf(w + r);
#pragma unroll
        for (int t = 0; t < kAbsTok; ++t) acc[t] = fmaf(sm[t * R + r], wv, acc[t]);
      }
    }
#pragma unroll
    for (int t = 0; t < kAbsTok; ++t) {
      float s = warp_sum(acc[t]);
      if (lane == t && t < cnt) {
        if (gate != nullptr) s *= sigmoid_f(ldf(gate + (n0 + t) * ldg + h * dv + v));
        stf(o + (static_cast<int64_t>(n0 + t) * H + h) * dv + v, s);
      }
    }
  }
}

// o *= sigmoid(gate), rows of N features; kVec: a 16-byte vector of features per thread and step.
template <typename T, bool kVec>
__global__ void __launch_bounds__(256)
sigmoid_gate_kernel(T* __restrict__ o, const T* __restrict__ gate, int64_t ldg, int64_t total, int N) {
  constexpr int V = kVec ? Vec16<T>::n : 1;
  for (int64_t i = (static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x) * V; i < total;
       i += static_cast<int64_t>(gridDim.x) * blockDim.x * V) {
    const T* g = gate + i / N * ldg + i % N;
    if constexpr (kVec) {
      float a[V], b[V];
      Vec16<T>::load(o + i, a);
      Vec16<T>::load(g, b);
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] *= sizeof(T) == 2 ? sigmoid_approx(b[j]) : sigmoid_f(b[j]);
      if constexpr (sizeof(T) == 2)
        *reinterpret_cast<uint4*>(o + i) = make_uint4(pack_bf16x2(a[0], a[1]), pack_bf16x2(a[2], a[3]), pack_bf16x2(a[4], a[5]), pack_bf16x2(a[6], a[7]));
      else
        *reinterpret_cast<float4*>(o + i) = make_float4(a[0], a[1], a[2], a[3]);
    } else {
      stf(o + i, ldf(o + i) * sigmoid_f(ldf(g)));
    }
  }
}

// Latent attention, any sizes. The heads of a token share the cached rows, so the work items of a sequence are its
// (token, head) pairs with the head running fastest; a block owns kLaQ consecutive pairs and walks the keys in tiles of
// 32 rows staged in shared memory as fp32. Warp w scores pairs w and w + 4 with one key per lane, keeps their running
// maxima and sums and accumulates their outputs in shared memory.
constexpr int kLaQ = 8, kLaK = 32, kLaWarps = 4, kLaMine = kLaQ / kLaWarps;

template <typename T>
__global__ void __launch_bounds__(kLaWarps * 32)
latent_attn_kernel(const SeqBatch sb, const T* __restrict__ qf, const PagedRows pages, int R,
                   const float* __restrict__ sink, float scale, int window, int H, float* __restrict__ part_o,
                   float* __restrict__ part_ml, T* __restrict__ o_lat) {
  extern __shared__ float sm[];
  const int W = pages.width, WS = W | 1;   // odd stride: lanes read a column of keys without bank conflicts
  float* sk = sm;                          // [kLaK][WS]
  float* sq = sk + kLaK * WS;              // [kLaQ][W]
  float* so = sq + kLaQ * W;               // [kLaQ][R]
  float* sp = so + kLaQ * R;               // [kLaQ][kLaK]
  const int split = blockIdx.y, S = gridDim.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // tile -> (sequence, first pair)
  int tile = blockIdx.x, b = 0, r0 = -1, cnt = 0;
  for (; b < sb.n_seq; ++b) {
    const int pairs = (sb.cu[b + 1] - sb.cu[b]) * H, tiles = (pairs + kLaQ - 1) / kLaQ;
    if (tile < tiles) {
      r0 = tile * kLaQ;
      cnt = min(kLaQ, pairs - r0);
      break;
    }
    tile -= tiles;
  }
  if (r0 < 0) return;
  const int slot = sb.ids[b], start = sb.start[b];
  const int64_t g0 = static_cast<int64_t>(sb.cu[b]) * H + r0;   // first pair in the packed arrays
  const int n_keys = start + (r0 + cnt - 1) / H + 1;
  const int tile0 = max(0, start + r0 / H - window + 1) / kLaK;   // from the window of the first query on
  const int tiles_k = (n_keys + kLaK - 1) / kLaK, per = (tiles_k - tile0 + S - 1) / S;
  const int kt0 = tile0 + split * per, kt1 = min(tiles_k, kt0 + per);
  for (int i = threadIdx.x; i < kLaQ * W; i += blockDim.x) sq[i] = i < cnt * W ? ldf(qf + g0 * W + i) : 0.f;
  for (int i = threadIdx.x; i < kLaQ * R; i += blockDim.x) so[i] = 0.f;
  float m[kLaMine], l[kLaMine];
  int pos[kLaMine];                        // position of the pair's token; -1: no pair
#pragma unroll
  for (int j = 0; j < kLaMine; ++j) {
    const int q = warp + j * kLaWarps;
    m[j] = -INFINITY;
    l[j] = 0.f;
    pos[j] = q < cnt ? start + (r0 + q) / H : -1;
  }
  for (int kt = kt0; kt < kt1; ++kt) {
    __syncthreads();
    for (int k = warp; k < kLaK; k += kLaWarps) {
      const int p = kt * kLaK + k;
      const int64_t row = p < n_keys ? page_row(pages, slot, p) : -1;
      const T* src = static_cast<const T*>(pages.pool) + (row < 0 ? 0 : row) * W;
      if (row >= 0 && W % Vec16<T>::n == 0) {
        for (int i = lane * Vec16<T>::n; i < W; i += 32 * Vec16<T>::n) {
          float f[Vec16<T>::n];
          Vec16<T>::load(src + i, f);
#pragma unroll
          for (int j = 0; j < Vec16<T>::n; ++j) sk[k * WS + i + j] = f[j];
        }
      } else {
        for (int i = lane; i < W; i += 32) sk[k * WS + i] = row < 0 ? 0.f : ldf(src + i);
      }
    }
    __syncthreads();
    float s[kLaMine];
#pragma unroll
    for (int j = 0; j < kLaMine; ++j) s[j] = 0.f;
    const float* kv = sk + lane * WS;
    const float* qv = sq + warp * W;
#pragma unroll 4
    for (int i = 0; i < W; ++i) {
      const float kk = kv[i];
#pragma unroll
      for (int j = 0; j < kLaMine; ++j) s[j] = fmaf(qv[j * kLaWarps * W + i], kk, s[j]);
    }
    float a[kLaMine];
#pragma unroll
    for (int j = 0; j < kLaMine; ++j) {
      const int kp = kt * kLaK + lane;
      const float sc = kp <= pos[j] && pos[j] - kp < window ? s[j] * scale : -INFINITY;
      const float mn = fmaxf(m[j], warp_max(sc));
      const float ref = mn == -INFINITY ? 0.f : mn;   // nothing seen yet: every weight below is 0
      const float p = expf(sc - ref);
      a[j] = expf(m[j] - ref);
      l[j] = l[j] * a[j] + warp_sum(p);
      m[j] = mn;
      sp[(warp + j * kLaWarps) * kLaK + lane] = p;
    }
    __syncwarp();
    for (int c = lane; c < R; c += 32) {
      float o[kLaMine];
#pragma unroll
      for (int j = 0; j < kLaMine; ++j) o[j] = so[(warp + j * kLaWarps) * R + c] * a[j];
#pragma unroll 8
      for (int k = 0; k < kLaK; ++k) {
        const float v = sk[k * WS + c];
#pragma unroll
        for (int j = 0; j < kLaMine; ++j) o[j] = fmaf(sp[(warp + j * kLaWarps) * kLaK + k], v, o[j]);
      }
#pragma unroll
      for (int j = 0; j < kLaMine; ++j) so[(warp + j * kLaWarps) * R + c] = o[j];
    }
  }
#pragma unroll
  for (int j = 0; j < kLaMine; ++j) {
    const int q = warp + j * kLaWarps;
    if (q >= cnt) continue;
    const int64_t nh = g0 + q;
    if (S == 1) {
      const int h = (r0 + q) % H;
      float mm = m[j];
      if (sink != nullptr) mm = fmaxf(mm, sink[h]);
      const float f = expf(m[j] - mm);
      float den = l[j] * f;
      if (sink != nullptr) den += expf(sink[h] - mm);
      const float w = f / den;
      for (int c = lane; c < R; c += 32) stf(o_lat + nh * R + c, so[q * R + c] * w);
    } else {
      for (int c = lane; c < R; c += 32) part_o[(nh * S + split) * R + c] = so[q * R + c];
      if (lane == 0) {
        part_ml[(nh * S + split) * 2] = m[j];
        part_ml[(nh * S + split) * 2 + 1] = l[j];
      }
    }
  }
}

template <typename T>
__global__ void latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                    const float* __restrict__ sink, int H, int R, int S, T* __restrict__ o_lat) {
  const int64_t nh = blockIdx.x;
  const float sk = sink != nullptr ? sink[nh % H] : -INFINITY;
  float mm = sk;
  for (int s = 0; s < S; ++s) mm = fmaxf(mm, part_ml[(nh * S + s) * 2]);
  float den = sink != nullptr ? expf(sk - mm) : 0.f;
  for (int s = 0; s < S; ++s) den += part_ml[(nh * S + s) * 2 + 1] * expf(part_ml[(nh * S + s) * 2] - mm);
  for (int c = threadIdx.x; c < R; c += blockDim.x) {
    float v = 0.f;
    for (int s = 0; s < S; ++s) {
      const float ms = part_ml[(nh * S + s) * 2];
      if (ms != -INFINITY) v += part_o[(nh * S + s) * R + c] * expf(ms - mm);
    }
    stf(o_lat + nh * R + c, v / den);
  }
}

// ---- experts -----------------------------------------------------------------------------------------------------
__device__ __forceinline__ float clamped_glu(float g, float u, const GluArgs& a) {
  g = fminf(g, a.limit);
  u = fminf(fmaxf(u, -a.limit), a.limit);
  return g * sigmoid_f(a.alpha * g) * (u + a.shift);
}

// The next expert in order of falling logits (equal ones by index) after expert `pi` with logit `pv`; -1: none left.
// Called by a whole warp with uniform arguments; every lane gets the result.
__device__ __forceinline__ int next_best(const float* z, int E, float pv, int pi, float& value) {
  float bv = -INFINITY;
  int bi = -1;
  for (int i = threadIdx.x & 31; i < E; i += 32) {
    const float v = z[i];
    if ((v < pv || (v == pv && i > pi)) && (bi < 0 || v > bv)) { bv = v; bi = i; }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (oi >= 0 && (bi < 0 || ov > bv || (ov == bv && oi < bi))) { bv = ov; bi = oi; }
  }
  value = bv;
  return bi;
}

// Experts of token m into `chosen` (shared memory, c.top entries, -1: bad token or table entry), scores' logits into
// `score` when that is not null; `z` holds c.E floats of shared memory for the router. The whole block calls it. Ranks are
// counted, one logit per thread: no chain of reductions.
__device__ __forceinline__ void choose_experts(const ExpertChoice& c, int m, float* z, int* chosen, float* score) {
  for (int j = threadIdx.x; j < c.top; j += blockDim.x) {
    const int tok = c.logits == nullptr ? c.tokens[m] : -1;
    chosen[j] = tok >= 0 && tok < c.vocab ? c.table[static_cast<int64_t>(tok) * c.top + j] : -1;
  }
  if (c.logits != nullptr) {
    const int pad = (c.E + 3) & ~3;
    for (int i = threadIdx.x; i < pad; i += blockDim.x) z[i] = i < c.E ? c.logits[static_cast<int64_t>(m) * c.E + i] : -INFINITY;
    __syncthreads();
    for (int i = threadIdx.x; i < c.E; i += blockDim.x) {
      const float v = z[i];
      int rank = 0;
#pragma unroll 4
      for (int k = 0; k < pad; k += 4) {
        const float4 o = *reinterpret_cast<const float4*>(z + k);
        rank += (o.x > v || (o.x == v && k < i)) + (o.y > v || (o.y == v && k + 1 < i)) + (o.z > v || (o.z == v && k + 2 < i)) +
                (o.w > v || (o.w == v && k + 3 < i));
      }
      if (rank < c.top && v == v) {
        chosen[rank] = i;
        if (score != nullptr) score[rank] = v;
      }
    }
  }
  __syncthreads();
}
// shared memory of choose_experts: logits, then experts, then scores
__host__ __device__ __forceinline__ int choice_smem(const ExpertChoice& c) {
  return 4 * ((c.logits != nullptr ? (c.E + 3) & ~3 : 0) + 2 * c.top);
}

// One warp per token: ids and sigmoid scores of the `top` largest logits.
__global__ void sigmoid_topk_kernel(const ExpertChoice c, int M, int* __restrict__ ids, float* __restrict__ weights, int* status) {
  const int m = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (m >= M) return;
  const float* z = c.logits + static_cast<int64_t>(m) * c.E;
  float v = INFINITY;
  int e = -1;
  for (int j = 0; j < c.top; ++j) {
    if (j == 0 || e >= 0) e = next_best(z, c.E, v, e, v);
    if ((threadIdx.x & 31) == 0) {
      if (e < 0) report_status(status, kBadArgument, 304, m, j);
      ids[static_cast<int64_t>(m) * c.top + j] = e < 0 ? 0 : e;          // never past the expert table
      weights[static_cast<int64_t>(m) * c.top + j] = e < 0 ? 0.f : sigmoid_f(v);
    }
  }
}

constexpr int kExpWarps = 8;

// h[m * top + j, i] = glu(w gate_e[i] . x[m], w up_e[i] . x[m]) with the token's j-th expert e and its input factor w;
// w_gate_up [E, 2 I, D].
template <typename T, bool kVec>
__global__ void __launch_bounds__(kExpWarps * 32)
experts_up_kernel(const T* __restrict__ x, const ExpertChoice c, const T* __restrict__ w, GluArgs glu, T* __restrict__ h, int D,
                  int I, int* status) {
  extern __shared__ __align__(16) float zs[];
  const int pair = blockIdx.x, m = pair / c.top;
  int* chosen = reinterpret_cast<int*>(zs + (choice_smem(c) / 4 - 2 * c.top));
  float* score = reinterpret_cast<float*>(chosen + c.top);
  choose_experts(c, m, zs, chosen, score);
  const int e = chosen[pair % c.top];
  const float wt = c.logits != nullptr ? sigmoid_f(score[pair % c.top]) : 1.f;
  if (e < 0 || e >= c.E) {
    if (threadIdx.x == 0) report_status(status, kBadArgument, 303, m, e);
    return;
  }
  const int lane = threadIdx.x & 31;
  const T* xr = x + static_cast<int64_t>(m) * D;
  for (int i = blockIdx.y * kExpWarps + (threadIdx.x >> 5); i < I; i += gridDim.y * kExpWarps) {
    const T* wg = w + (static_cast<int64_t>(e) * 2 * I + i) * D;
    const T* wu = wg + static_cast<int64_t>(I) * D;
    float g = 0.f, u = 0.f;
    if constexpr (kVec) {
      constexpr int V = Vec16<T>::n;
#pragma unroll 4
      for (int k = lane * V; k < D; k += 32 * V) {
        float xv[V], gv[V], uv[V];
        Vec16<T>::load(xr + k, xv);
        Vec16<T>::load(wg + k, gv);
        Vec16<T>::load(wu + k, uv);
#pragma unroll
        for (int j = 0; j < V; ++j) {
          g = fmaf(xv[j], gv[j], g);
          u = fmaf(xv[j], uv[j], u);
        }
      }
    } else {
      for (int k = lane; k < D; k += 32) {
        const float xv = ldf(xr + k);
        g = fmaf(xv, ldf(wg + k), g);
        u = fmaf(xv, ldf(wu + k), u);
      }
    }
    g = warp_sum(g);
    u = warp_sum(u);
    if (lane == 0) stf(h + static_cast<int64_t>(pair) * I + i, clamped_glu(wt * g, wt * u, glu));
  }
}

// x[m, d] += out_scale * sum_j down_e(j)[d] . h[m * top + j]; w_down [E, D, I]. A warp owns an output feature and walks its
// experts' rows kJ at a time (few rows: two, for more loads in flight; more rows: one, for more blocks).
template <typename T, bool kVec, int kJ>
__global__ void __launch_bounds__(kExpWarps * 32)
experts_down_kernel(const T* __restrict__ h, const ExpertChoice c, const T* __restrict__ w, float out_scale, float* __restrict__ x,
                    int D, int I) {
  extern __shared__ __align__(16) float zs[];
  const int m = blockIdx.x, lane = threadIdx.x & 31;
  int* chosen = reinterpret_cast<int*>(zs + (choice_smem(c) / 4 - 2 * c.top));
  choose_experts(c, m, zs, chosen, nullptr);
  const T* hm = h + static_cast<int64_t>(m) * c.top * I;
  for (int d = blockIdx.y * kExpWarps + (threadIdx.x >> 5); d < D; d += gridDim.y * kExpWarps) {
    float* xo = x + static_cast<int64_t>(m) * D + d;
    const float before = *xo;
    float acc = 0.f;
    for (int j = 0; j < c.top; j += kJ) {
      const T *wr[kJ], *hr[kJ];
      bool ok[kJ];
      float part[kJ];
#pragma unroll
      for (int q = 0; q < kJ; ++q) {   // a missing expert reads its neighbour's rows (or expert 0's) and counts nothing
        const int e = j + q < c.top ? chosen[j + q] : -1;
        ok[q] = e >= 0 && e < c.E;
        wr[q] = w + (static_cast<int64_t>(ok[q] ? e : 0) * D + d) * I;
        hr[q] = hm + static_cast<int64_t>(ok[q] ? j + q : 0) * I;
        part[q] = 0.f;
      }
      if constexpr (kVec) {
        constexpr int V = Vec16<T>::n;
#pragma unroll 4
        for (int k = lane * V; k < I; k += 32 * V) {
#pragma unroll
          for (int q = 0; q < kJ; ++q) {
            float hv[V], wv[V];
            Vec16<T>::load(hr[q] + k, hv);
            Vec16<T>::load(wr[q] + k, wv);
#pragma unroll
            for (int t = 0; t < V; ++t) part[q] = fmaf(hv[t], wv[t], part[q]);
          }
        }
      } else {
        for (int k = lane; k < I; k += 32)
#pragma unroll
          for (int q = 0; q < kJ; ++q) part[q] = fmaf(ldf(hr[q] + k), ldf(wr[q] + k), part[q]);
      }
#pragma unroll
      for (int q = 0; q < kJ; ++q) acc += ok[q] ? part[q] : 0.f;
    }
    acc = warp_sum(acc);
    if (lane == 0) *xo = before + acc * out_scale;
  }
}

__global__ void moe_gather_rows_kernel(const __nv_bfloat16* __restrict__ x, const int* __restrict__ idx,
                                       const int* __restrict__ pos, const int* __restrict__ offs_end,
                                       const int* __restrict__ counts, const float* __restrict__ w_pair, int top,
                                       __nv_bfloat16* __restrict__ xs, int* __restrict__ row_of, float* __restrict__ w_row, int D) {
  const int p = blockIdx.x, e = idx[p];
  const int row = offs_end[e] - counts[e] + pos[p];
  if (threadIdx.x == 0) {
    row_of[p] = row;
    if (w_pair != nullptr) w_row[row] = w_pair[p];
  }
  const uint4* src = reinterpret_cast<const uint4*>(x + static_cast<int64_t>(p / top) * D);
  uint4* dst = reinterpret_cast<uint4*>(xs + static_cast<int64_t>(row) * D);
  for (int i = threadIdx.x; i < D / 8; i += blockDim.x) dst[i] = src[i];
}

__global__ void clamped_glu_kernel(const __nv_bfloat16* __restrict__ gu, const float* __restrict__ w_row, GluArgs glu,
                                   __nv_bfloat16* __restrict__ h, int64_t n8, int I8) {
  for (int64_t i = blockIdx.x * static_cast<int64_t>(blockDim.x) + threadIdx.x; i < n8;
       i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t r = i / I8, c = i % I8;
    const float w = w_row != nullptr ? w_row[r] : 1.f;
    float g[8], u[8];
    Vec16<__nv_bfloat16>::load(gu + (r * 2 * I8 + c) * 8, g);
    Vec16<__nv_bfloat16>::load(gu + (r * 2 * I8 + I8 + c) * 8, u);
    uint32_t o[4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
      o[j] = pack_bf16x2(clamped_glu(w * g[2 * j], w * u[2 * j], glu), clamped_glu(w * g[2 * j + 1], w * u[2 * j + 1], glu));
    *reinterpret_cast<uint4*>(h + i * 8) = make_uint4(o[0], o[1], o[2], o[3]);
  }
}

__global__ void moe_combine_rows_kernel(const __nv_bfloat16* __restrict__ ys, const int* __restrict__ row_of, int top,
                                        float w, float* __restrict__ x, int D) {
  const int m = blockIdx.x;
  float* xr = x + static_cast<int64_t>(m) * D;
  for (int i = threadIdx.x; i < D / 8; i += blockDim.x) {
    float acc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = 0.f;
    for (int t = 0; t < top; ++t) {
      float v[8];
      Vec16<__nv_bfloat16>::load(ys + static_cast<int64_t>(row_of[m * top + t]) * D + i * 8, v);
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] += v[j];
    }
    float4* xp = reinterpret_cast<float4*>(xr + i * 8);
    float4 a = xp[0], c = xp[1];
    a.x += w * acc[0]; a.y += w * acc[1]; a.z += w * acc[2]; a.w += w * acc[3];
    c.x += w * acc[4]; c.y += w * acc[5]; c.z += w * acc[6]; c.w += w * acc[7];
    xp[0] = a;
    xp[1] = c;
  }
}

int threads_for(int n) { return n >= 1024 ? 256 : (n >= 256 ? 128 : 64); }

template <typename T>
cudaError_t latent_attention_t(const SeqBatch& sb, const T* qf, const PagedRows& pages, int R, const float* sink, float scale,
                               int window, int H, int n_splits, float* part_o, float* part_ml, T* o_lat, cudaStream_t st) {
  static int have = 0;
  const int smem = 4 * (kLaK * (pages.width + 1) + kLaQ * pages.width + kLaQ * R + kLaQ * kLaK);
  cudaError_t e = want_smem(latent_attn_kernel<T>, smem, have);
  if (e != cudaSuccess) return e;
  const dim3 grid(static_cast<unsigned>(static_cast<int64_t>(sb.n_tok) * H / kLaQ + sb.n_seq), n_splits);
  latent_attn_kernel<T><<<grid, kLaWarps * 32, smem, st>>>(sb, qf, pages, R, sink, scale, window, H, part_o, part_ml, o_lat);
  if (n_splits > 1) latent_merge_kernel<T><<<sb.n_tok * H, 128, 0, st>>>(part_o, part_ml, sink, H, R, n_splits, o_lat);
  return cudaGetLastError();
}

template <typename T>
cudaError_t absorb_q_t(const SeqBatch& sb, const T* q, int64_t ldq, const T* w_uk, T* qf, int H, int dn, int dr, int R,
                       const RopeTable& rope, cudaStream_t st) {
  static int have_v = 0, have_s = 0;
  const int smem = 4 * (kAbsTok * (dn + dr) + 8 * kAbsTok * kAbsCols);
  const bool vec = R % 8 == 0 && (reinterpret_cast<uintptr_t>(w_uk) & 15) == 0;
  cudaError_t e = vec ? want_smem(mla_absorb_q_kernel<T, true>, smem, have_v) : want_smem(mla_absorb_q_kernel<T, false>, smem, have_s);
  if (e != cudaSuccess) return e;
  const dim3 grid((sb.n_tok + kAbsTok - 1) / kAbsTok, H, (R + kAbsCols - 1) / kAbsCols);
  if (vec) mla_absorb_q_kernel<T, true><<<grid, 256, smem, st>>>(sb, q, ldq, w_uk, qf, H, dn, dr, R, rope);
  else mla_absorb_q_kernel<T, false><<<grid, 256, smem, st>>>(sb, q, ldq, w_uk, qf, H, dn, dr, R, rope);
  return cudaGetLastError();
}

template <typename T>
cudaError_t absorb_out_t(const T* o_lat, const T* w_uv, const T* gate, int64_t ldg, T* o, int n_tok, int H, int dv, int R, cudaStream_t st) {
  static int have_v = 0, have_s = 0;
  const int smem = 4 * kAbsTok * R;
  const bool vec = R % Vec16<T>::n == 0 && ((reinterpret_cast<uintptr_t>(w_uv) | reinterpret_cast<uintptr_t>(o_lat)) & 15) == 0;
  cudaError_t e = vec ? want_smem(mla_absorb_out_kernel<T, true>, smem, have_v) : want_smem(mla_absorb_out_kernel<T, false>, smem, have_s);
  if (e != cudaSuccess) return e;
  const int tiles = (n_tok + kAbsTok - 1) / kAbsTok;
  const int per = (dv + 7) / 8, z = tiles * H < 148 ? (per < 16 ? per : 16) : 1;
  const dim3 grid(tiles, H, z);
  if (vec) mla_absorb_out_kernel<T, true><<<grid, 256, smem, st>>>(o_lat, w_uv, gate, ldg, o, n_tok, H, dv, R);
  else mla_absorb_out_kernel<T, false><<<grid, 256, smem, st>>>(o_lat, w_uv, gate, ldg, o, n_tok, H, dv, R);
  return cudaGetLastError();
}

}  // namespace

cudaError_t launch_seq_begin(const int* ids, const int* cu, const int* tokens, int n_seq, int max_slots, int* lens,
                             int* prev, int* start, int* prev_tok, int* status, cudaStream_t st) {
  seq_begin_kernel<<<(n_seq + 63) / 64, 64, 0, st>>>(ids, cu, tokens, n_seq, max_slots, lens, prev, start, prev_tok, status);
  return cudaGetLastError();
}

cudaError_t launch_embed_bigram(bool f32, const SeqBatch& sb, const int* tokens, const int* prev_tok, const void* embed,
                                int vocab, const void* bigram, long long buckets, long long mul_prev, long long mul_cur,
                                int D, float* x, int* status, cudaStream_t st) {
  if (f32)
    embed_bigram_kernel<float><<<sb.n_tok, threads_for(D), 0, st>>>(sb, tokens, prev_tok, static_cast<const float*>(embed), vocab,
                                                                    static_cast<const float*>(bigram), buckets, mul_prev,
                                                                    mul_cur, D, x, status);
  else
    embed_bigram_kernel<__nv_bfloat16><<<sb.n_tok, threads_for(D), 0, st>>>(
        sb, tokens, prev_tok, static_cast<const __nv_bfloat16*>(embed), vocab, static_cast<const __nv_bfloat16*>(bigram),
        buckets, mul_prev, mul_cur, D, x, status);
  return cudaGetLastError();
}

cudaError_t launch_norm_rows(bool f32_out, int mode, const float* x, const float* gamma, const float* beta, void* out,
                             int rows, int D, float eps, cudaStream_t st) {
  if (f32_out) norm_rows_go(mode, x, gamma, beta, static_cast<float*>(out), rows, D, eps, st);
  else norm_rows_go(mode, x, gamma, beta, static_cast<__nv_bfloat16*>(out), rows, D, eps, st);
  return cudaGetLastError();
}

cudaError_t launch_residual_norm(bool y_f32, bool f32_out, const void* y, const float* gpost, float* x, bool add,
                                 const float* gnext, void* out, int rows, int D, float eps, cudaStream_t st) {
  const float* yf = static_cast<const float*>(y);
  const __nv_bfloat16* yb = static_cast<const __nv_bfloat16*>(y);
  if (f32_out) {
    if (!y_f32) return cudaErrorInvalidValue;
    residual_norm_go(yf, gpost, x, add, gnext, static_cast<float*>(out), rows, D, eps, st);
  } else if (y_f32) {
    residual_norm_go(yf, gpost, x, add, gnext, static_cast<__nv_bfloat16*>(out), rows, D, eps, st);
  } else {
    residual_norm_go(yb, gpost, x, add, gnext, static_cast<__nv_bfloat16*>(out), rows, D, eps, st);
  }
  return cudaGetLastError();
}

cudaError_t launch_rows_linear(bool f32, const void* x, int64_t ldx, const void* w, int64_t ldw, int M, int N, int K,
                               const RowsOut& out, cudaStream_t st) {
  if (M < 1 || N < 1 || K < 1 || (out.n1 < N && out.y2 == nullptr)) return cudaErrorInvalidValue;
  if (out.act == kActSiluGlu)
    return f32 ? rows_linear_t<float, true>(x, ldx, w, ldw, M, N, K, out, st)
               : rows_linear_t<__nv_bfloat16, true>(x, ldx, w, ldw, M, N, K, out, st);
  return f32 ? rows_linear_t<float, false>(x, ldx, w, ldw, M, N, K, out, st)
             : rows_linear_t<__nv_bfloat16, false>(x, ldx, w, ldw, M, N, K, out, st);
}

cudaError_t launch_mla_prepare(bool f32, const SeqBatch& sb, const void* y, int64_t ldy, int q_rank, int R, int dr,
                               const float* q_gamma, const float* kv_gamma, float eps, const RopeTable& rope,
                               const PagedRows& pages, void* cq, void* lat, int* status, cudaStream_t st) {
  const int th = threads_for(q_rank + R + dr);
#define B200_MLA(T, HOLD)                                                                                                                       \
  mla_prepare_kernel<T, HOLD><<<sb.n_tok, th, 0, st>>>(sb, static_cast<const T*>(y), ldy, q_rank, R, dr, q_gamma, kv_gamma, eps, rope, pages, \
                                                       static_cast<T*>(cq), static_cast<T*>(lat), status)
  if (sb.n_tok <= 64) { if (f32) B200_MLA(float, 8); else B200_MLA(__nv_bfloat16, 8); }
  else { if (f32) B200_MLA(float, 0); else B200_MLA(__nv_bfloat16, 0); }
#undef B200_MLA
  return cudaGetLastError();
}

cudaError_t launch_mla_rope_qk(bool f32, const SeqBatch& sb, void* q, int64_t ldq, const void* kn, int64_t ldkn, const void* lat,
                               int64_t ldlat, int R, void* k, int H, int dn, int dr, const RopeTable& rope, cudaStream_t st) {
  if (f32)
    mla_rope_qk_kernel<float><<<sb.n_tok, 256, 0, st>>>(sb, static_cast<float*>(q), ldq, static_cast<const float*>(kn), ldkn,
                                                        static_cast<const float*>(lat), ldlat, R, static_cast<float*>(k), H, dn, dr, rope);
  else
    mla_rope_qk_kernel<__nv_bfloat16><<<sb.n_tok, 256, 0, st>>>(
        sb, static_cast<__nv_bfloat16*>(q), ldq, static_cast<const __nv_bfloat16*>(kn), ldkn, static_cast<const __nv_bfloat16*>(lat),
        ldlat, R, static_cast<__nv_bfloat16*>(k), H, dn, dr, rope);
  return cudaGetLastError();
}

cudaError_t launch_mla_absorb_q(bool f32, const SeqBatch& sb, const void* q, int64_t ldq, const void* w_uk, void* qf, int H, int dn,
                                int dr, int R, const RopeTable& rope, cudaStream_t st) {
  return f32 ? absorb_q_t<float>(sb, static_cast<const float*>(q), ldq, static_cast<const float*>(w_uk), static_cast<float*>(qf), H, dn,
                                 dr, R, rope, st)
             : absorb_q_t<__nv_bfloat16>(sb, static_cast<const __nv_bfloat16*>(q), ldq, static_cast<const __nv_bfloat16*>(w_uk),
                                         static_cast<__nv_bfloat16*>(qf), H, dn, dr, R, rope, st);
}

cudaError_t launch_mla_absorb_out(bool f32, const void* o_lat, const void* w_uv, const void* gate, int64_t ldg, void* o, int n_tok, int H,
                                  int dv, int R, cudaStream_t st) {
  return f32 ? absorb_out_t<float>(static_cast<const float*>(o_lat), static_cast<const float*>(w_uv), static_cast<const float*>(gate), ldg,
                                   static_cast<float*>(o), n_tok, H, dv, R, st)
             : absorb_out_t<__nv_bfloat16>(static_cast<const __nv_bfloat16*>(o_lat), static_cast<const __nv_bfloat16*>(w_uv),
                                           static_cast<const __nv_bfloat16*>(gate), ldg, static_cast<__nv_bfloat16*>(o), n_tok, H, dv, R, st);
}

cudaError_t launch_sigmoid_gate(bool f32, void* o, const void* gate, int64_t ldg, int rows, int N, cudaStream_t st) {
  const int V = f32 ? 4 : 8;
  const bool vec = N % V == 0 && ldg % V == 0 && ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate)) & 15) == 0;
  const int64_t total = static_cast<int64_t>(rows) * N, blocks = (total / (vec ? V : 1) + 255) / 256;
  const int grid = static_cast<int>(blocks < 148 * 16 ? (blocks < 1 ? 1 : blocks) : 148 * 16);
#define B200_GATE(T, K) sigmoid_gate_kernel<T, K><<<grid, 256, 0, st>>>(static_cast<T*>(o), static_cast<const T*>(gate), ldg, total, N)
  if (f32) { if (vec) B200_GATE(float, true); else B200_GATE(float, false); }
  else { if (vec) B200_GATE(__nv_bfloat16, true); else B200_GATE(__nv_bfloat16, false); }
#undef B200_GATE
  return cudaGetLastError();
}

cudaError_t launch_latent_attention(bool f32, const SeqBatch& sb, const void* qf, const PagedRows& pages, int R,
                                    const float* sink, float scale, int window, int H, int n_splits, float* part_o, float* part_ml,
                                    void* o_lat, cudaStream_t st) {
  if (window < 1 || n_splits < 1 || (n_splits > 1 && (part_o == nullptr || part_ml == nullptr))) return cudaErrorInvalidValue;
  return f32 ? latent_attention_t<float>(sb, static_cast<const float*>(qf), pages, R, sink, scale, window, H, n_splits, part_o, part_ml,
                                         static_cast<float*>(o_lat), st)
             : latent_attention_t<__nv_bfloat16>(sb, static_cast<const __nv_bfloat16*>(qf), pages, R, sink, scale, window, H, n_splits,
                                                 part_o, part_ml, static_cast<__nv_bfloat16*>(o_lat), st);
}

cudaError_t launch_experts_up(bool f32, const void* x, const ExpertChoice& c, const void* w, GluArgs glu, void* h, int M, int D,
                              int I, int* status, cudaStream_t st) {
  // enough blocks for the loads in flight, few enough that the choice of the experts is not repeated too often
  const int per = (I + kExpWarps - 1) / kExpWarps, want = 148 * (M <= 2 ? 16 : 8) / (M * c.top), smem = choice_smem(c);
  const dim3 grid(M * c.top, want < 1 ? 1 : (want < per ? want : per));
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  const bool vec = D % (f32 ? 4 : 8) == 0;
#define B200_UP(T, V) \
  experts_up_kernel<T, V><<<grid, kExpWarps * 32, smem, st>>>(static_cast<const T*>(x), c, static_cast<const T*>(w), glu, static_cast<T*>(h), D, I, status)
  if (f32) { if (vec) B200_UP(float, true); else B200_UP(float, false); }
  else { if (vec) B200_UP(__nv_bfloat16, true); else B200_UP(__nv_bfloat16, false); }
#undef B200_UP
  return cudaGetLastError();
}

cudaError_t launch_experts_down(bool f32, const void* h, const ExpertChoice& c, const void* w, float out_scale, float* x, int M,
                                int D, int I, cudaStream_t st) {
  const int per = (D + kExpWarps - 1) / kExpWarps, want = 148 * 16 / M, smem = choice_smem(c);
  const dim3 grid(M, want < 1 ? 1 : (want < per ? want : per));
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  const bool vec = I % (f32 ? 4 : 8) == 0;
#define B200_DN(T, V) \
  {                                                                                                                                         \
    if (M <= 2) experts_down_kernel<T, V, 2><<<grid, kExpWarps * 32, smem, st>>>(static_cast<const T*>(h), c, static_cast<const T*>(w), out_scale, x, D, I); \
    else experts_down_kernel<T, V, 1><<<grid, kExpWarps * 32, smem, st>>>(static_cast<const T*>(h), c, static_cast<const T*>(w), out_scale, x, D, I);        \
  }
  if (f32) { if (vec) B200_DN(float, true) else B200_DN(float, false) }
  else { if (vec) B200_DN(__nv_bfloat16, true) else B200_DN(__nv_bfloat16, false) }
#undef B200_DN
  return cudaGetLastError();
}

cudaError_t launch_sigmoid_topk(const ExpertChoice& c, int M, int* ids, float* weights, int* status, cudaStream_t st) {
  if (c.top < 1 || c.top > c.E) return cudaErrorInvalidValue;
  sigmoid_topk_kernel<<<(M + 7) / 8, 256, 0, st>>>(c, M, ids, weights, status);
  return cudaGetLastError();
}

cudaError_t launch_moe_gather_rows(const __nv_bfloat16* x, const int* idx, const int* pos, const int* offs_end,
                                   const int* counts, const float* w_pair, int top, __nv_bfloat16* xs, int* row_of, float* w_row,
                                   int M, int D, cudaStream_t st) {
  if (D % 8 != 0) return cudaErrorInvalidValue;
  moe_gather_rows_kernel<<<M * top, 128, 0, st>>>(x, idx, pos, offs_end, counts, w_pair, top, xs, row_of, w_row, D);
  return cudaGetLastError();
}
cudaError_t launch_clamped_glu(const __nv_bfloat16* gu, const float* w_row, GluArgs glu, __nv_bfloat16* h, int rows, int I,
                               cudaStream_t st) {
  if (I % 8 != 0) return cudaErrorInvalidValue;
  const int64_t n8 = static_cast<int64_t>(rows) * (I / 8);
  const int grid = static_cast<int>((n8 + 255) / 256 < 148 * 16 ? (n8 + 255) / 256 : 148 * 16);
  clamped_glu_kernel<<<grid > 0 ? grid : 1, 256, 0, st>>>(gu, w_row, glu, h, n8, I / 8);
  return cudaGetLastError();
}
cudaError_t launch_moe_combine_rows(const __nv_bfloat16* ys, const int* row_of, int top, float w, float* x, int M, int D,
                                    cudaStream_t st) {
  if (D % 8 != 0) return cudaErrorInvalidValue;
  moe_combine_rows_kernel<<<M, 128, 0, st>>>(ys, row_of, top, w, x, D);
  return cudaGetLastError();
}

}  // namespace b200
