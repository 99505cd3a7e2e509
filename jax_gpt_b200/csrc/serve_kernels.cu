// Serving kernels of models whose layers run on packed (ragged) batches with a 32-bit residual: sequence
// bookkeeping, embedding plus bigram table, norms, few-row linear layers (decode), multi-head latent attention over
// paged latent rows (RMS-normed latents, interleaved rotary part, absorbed weights, softmax with a sink), and experts
// chosen by a token table with a clamped gated activation.
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

// ---- few-row linear ------------------------------------------------------------------------------------------------
constexpr int kLinWarps = 8;

__device__ __forceinline__ float row_act(float v, int act) {
  if (act == kActRelu2) {
    const float r = fmaxf(v, 0.f);
    return r * r;
  }
  return v;
}

// A warp computes NR output features for up to MR rows; lanes stride the contraction in 16-byte vectors.
template <typename T, int MR, int NR, bool kVec>
__global__ void __launch_bounds__(kLinWarps * 32)
rows_linear_kernel(const T* __restrict__ x, int64_t ldx, const T* __restrict__ w, int64_t ldw, void* __restrict__ y,
                   int64_t ldy, int M, int N, int K, int act, int out_mode) {
  const int lane = threadIdx.x & 31;
  const int n0 = (blockIdx.x * kLinWarps + (threadIdx.x >> 5)) * NR;
  const int m0 = blockIdx.y * MR;
  if (n0 >= N) return;
  float acc[MR][NR];
#pragma unroll
  for (int m = 0; m < MR; ++m)
#pragma unroll
    for (int r = 0; r < NR; ++r) acc[m][r] = 0.f;
  const T* wr[NR];
#pragma unroll
  for (int r = 0; r < NR; ++r) wr[r] = w + static_cast<int64_t>(n0 + r < N ? n0 + r : n0) * ldw;
  const T* xr[MR];
#pragma unroll
  for (int m = 0; m < MR; ++m) xr[m] = x + static_cast<int64_t>(m0 + m < M ? m0 + m : m0) * ldx;
  if constexpr (kVec) {
    constexpr int V = Vec16<T>::n;
#pragma unroll 2
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
  for (int m = 0; m < MR; ++m)
#pragma unroll
    for (int r = 0; r < NR; ++r)
      if (lane == ((m * NR + r) & 31) && m0 + m < M && n0 + r < N) {
        const float v = row_act(acc[m][r], act);
        const int64_t o = static_cast<int64_t>(m0 + m) * ldy + n0 + r;
        if (out_mode == 0) stf(static_cast<T*>(y) + o, v);
        else if (out_mode == 1) static_cast<float*>(y)[o] = v;
        else static_cast<float*>(y)[o] += v;
      }
}

template <typename T, int MR, int NR>
void rows_linear_go(bool vec, const T* x, int64_t ldx, const T* w, int64_t ldw, void* y, int64_t ldy, int M, int N, int K,
                    int act, int out_mode, cudaStream_t st) {
  const dim3 grid((N + kLinWarps * NR - 1) / (kLinWarps * NR), (M + MR - 1) / MR);
  if (vec)
    rows_linear_kernel<T, MR, NR, true><<<grid, kLinWarps * 32, 0, st>>>(x, ldx, w, ldw, y, ldy, M, N, K, act, out_mode);
  else
    rows_linear_kernel<T, MR, NR, false><<<grid, kLinWarps * 32, 0, st>>>(x, ldx, w, ldw, y, ldy, M, N, K, act, out_mode);
}

template <typename T>
cudaError_t rows_linear_t(const void* x, int64_t ldx, const void* w, int64_t ldw, void* y, int64_t ldy, int M, int N, int K,
                          int act, int out_mode, cudaStream_t st) {
  const bool vec = K % Vec16<T>::n == 0 && ldx % Vec16<T>::n == 0 && ldw % Vec16<T>::n == 0 &&
                   (reinterpret_cast<uintptr_t>(x) & 15) == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0;
  const T* xt = static_cast<const T*>(x);
  const T* wt = static_cast<const T*>(w);
  // narrow outputs take fewer features per warp so that the grid still covers the SMs
  const bool wide = N >= 148 * kLinWarps * 4;
#define B200_GO(MR)                                                                                       \
  (wide ? rows_linear_go<T, MR, 4>(vec, xt, ldx, wt, ldw, y, ldy, M, N, K, act, out_mode, st)             \
        : (N >= 148 * kLinWarps * 2 ? rows_linear_go<T, MR, 2>(vec, xt, ldx, wt, ldw, y, ldy, M, N, K, act, out_mode, st) \
                                    : rows_linear_go<T, MR, 1>(vec, xt, ldx, wt, ldw, y, ldy, M, N, K, act, out_mode, st)))
  if (M == 1) B200_GO(1);
  else if (M == 2) B200_GO(2);
  else if (M <= 4) B200_GO(4);
  else B200_GO(8);
#undef B200_GO
  return cudaGetLastError();
}

// ---- multi-head latent attention ------------------------------------------------------------------------------------
// Row of position `pos` of cache slot `slot` in a page pool, or -1.
__device__ __forceinline__ int64_t page_row(const PagedRows& pg, int slot, int pos) {
  const int pi = pos / pg.page_size;
  if (pi >= pg.max_pages) return -1;
  const int page = pg.block_table[static_cast<int64_t>(slot) * pg.max_pages + pi];
  if (page < 0 || page >= pg.n_pages) return -1;
  return static_cast<int64_t>(page) * pg.page_size + pos % pg.page_size;
}

// Feature i of a rotary part read through `at(i)`, turned to position `pos`.
template <typename F>
__device__ __forceinline__ float rotated(const RopeTable& r, int pos, int i, F at) {
  if (i >= r.dims) return at(i);
  const int64_t k = static_cast<int64_t>(pos) * (r.dims / 2) + (i >> 1);
  const float c = r.cos[k], s = r.sin[k];
  return (i & 1) == 0 ? at(i) * c - at(i + 1) * s : at(i) * c + at(i - 1) * s;
}

template <typename T>
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
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) { const float v = ldf(row + i); sq += v * v; }
  for (int i = threadIdx.x; i < R; i += blockDim.x) { const float v = ldf(kv + i); sk += v * v; }
  const float iq = 1.f / sqrtf(block_sum(sq, red) / q_rank + eps);
  const float ik = 1.f / sqrtf(block_sum(sk, red) / R + eps);
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x)
    stf(cq + static_cast<int64_t>(n) * q_rank + i, ldf(row + i) * iq * q_gamma[i]);
  const int64_t dst = page_row(pages, sb.ids[b], pos);
  if (dst < 0 || pos >= rope.max_pos) {
    if (threadIdx.x == 0) report_status(status, kBadArgument, 302, b, pos);
    return;
  }
  T* prow = static_cast<T*>(pages.pool) + dst * pages.width;
  T* lrow = lat != nullptr ? lat + static_cast<int64_t>(n) * (R + dr) : nullptr;
  for (int i = threadIdx.x; i < R + dr; i += blockDim.x) {
    float v;
    if (i < R) v = ldf(kv + i) * ik * kv_gamma[i];
    else v = rotated(rope, pos, i - R, [&](int j) { return ldf(kv + R + j); });
    stf(prow + i, v);
    if (lrow != nullptr) stf(lrow + i, v);
  }
}

// One block per token: query heads rotated in place, keys assembled.
template <typename T>
__global__ void mla_rope_qk_kernel(const SeqBatch sb, T* __restrict__ q, const T* __restrict__ kn, int64_t ldkn,
                                   const T* __restrict__ lat, int64_t ldlat, int R, T* __restrict__ k, int H, int dn, int dr,
                                   const RopeTable rope) {
  const int n = blockIdx.x;
  const int b = sb.tok_seq[n];
  const int pos = sb.start[b] + n - sb.cu[b];
  const int half = rope.dims / 2, D = dn + dr;
  T* qr = q + static_cast<int64_t>(n) * H * D;
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

constexpr int kAbsTok = 8;   // tokens per block of the absorption kernels

template <typename T>
__global__ void mla_absorb_q_kernel(const SeqBatch sb, const T* __restrict__ q, const T* __restrict__ w_uk,
                                    T* __restrict__ qf, int H, int dn, int dr, int R, const RopeTable rope) {
  extern __shared__ float sm[];   // [kAbsTok][dn + dr]
  const int D = dn + dr, h = blockIdx.y, n0 = blockIdx.x * kAbsTok;
  const int cnt = min(kAbsTok, sb.n_tok - n0);
  for (int i = threadIdx.x; i < cnt * D; i += blockDim.x)
    sm[i] = ldf(q + (static_cast<int64_t>(n0 + i / D) * H + h) * D + i % D);
  for (int i = threadIdx.x + cnt * D; i < kAbsTok * D; i += blockDim.x) sm[i] = 0.f;
  __syncthreads();
  const T* w = w_uk + static_cast<int64_t>(h) * dn * R;
  for (int r = blockIdx.z * blockDim.x + threadIdx.x; r < R; r += gridDim.z * blockDim.x) {
    float acc[kAbsTok];
#pragma unroll
    for (int t = 0; t < kAbsTok; ++t) acc[t] = 0.f;
#pragma unroll 4
    for (int d = 0; d < dn; ++d) {
      const float wv = ldf(w + static_cast<int64_t>(d) * R + r);
#pragma unroll
      for (int t = 0; t < kAbsTok; ++t) acc[t] = fmaf(sm[t * D + d], wv, acc[t]);
    }
    for (int t = 0; t < cnt; ++t) stf(qf + (static_cast<int64_t>(n0 + t) * H + h) * (R + dr) + r, acc[t]);
  }
  if (blockIdx.z == 0)
    for (int i = threadIdx.x; i < cnt * dr; i += blockDim.x) {
      const int t = i / dr, j = i % dr, n = n0 + t, b = sb.tok_seq[n];
      const int pos = sb.start[b] + n - sb.cu[b];
      stf(qf + (static_cast<int64_t>(n) * H + h) * (R + dr) + R + j,
          rotated(rope, min(pos, rope.max_pos - 1), j, [&](int k) { return sm[t * D + dn + k]; }));
    }
}

template <typename T>
__global__ void mla_absorb_out_kernel(const T* __restrict__ o_lat, const T* __restrict__ w_uv, T* __restrict__ o, int n_tok,
                                      int H, int dv, int R) {
  extern __shared__ float sm[];   // [kAbsTok][R]
  const int h = blockIdx.y, n0 = blockIdx.x * kAbsTok;
  const int cnt = min(kAbsTok, n_tok - n0);
  for (int i = threadIdx.x; i < cnt * R; i += blockDim.x)
    sm[i] = ldf(o_lat + (static_cast<int64_t>(n0 + i / R) * H + h) * R + i % R);
  for (int i = threadIdx.x + cnt * R; i < kAbsTok * R; i += blockDim.x) sm[i] = 0.f;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  for (int v = blockIdx.z * nw + warp; v < dv; v += gridDim.z * nw) {
    const T* w = w_uv + (static_cast<int64_t>(h) * dv + v) * R;
    float acc[kAbsTok];
#pragma unroll
    for (int t = 0; t < kAbsTok; ++t) acc[t] = 0.f;
#pragma unroll 4
    for (int r = lane; r < R; r += 32) {
      const float wv = ldf(w + r);
#pragma unroll
      for (int t = 0; t < kAbsTok; ++t) acc[t] = fmaf(sm[t * R + r], wv, acc[t]);
    }
#pragma unroll
    for (int t = 0; t < kAbsTok; ++t) {
      const float s = warp_sum(acc[t]);
      if (lane == t && t < cnt) stf(o + (static_cast<int64_t>(n0 + t) * H + h) * dv + v, s);
    }
  }
}

// Latent attention, any sizes. A block owns up to kLaQ consecutive queries of one sequence and one head; it walks
// the keys in tiles of 32 rows staged in shared memory as fp32. Warp w scores queries w, w + 4, ... with one key per
// lane and keeps their running maxima and sums; outputs are accumulated in shared memory.
constexpr int kLaQ = 8, kLaK = 32, kLaWarps = 4;

template <typename T>
__global__ void __launch_bounds__(kLaWarps * 32)
latent_attn_kernel(const SeqBatch sb, const T* __restrict__ qf, const PagedRows pages, int R,
                   const float* __restrict__ sink, float scale, int H, float* __restrict__ part_o,
                   float* __restrict__ part_ml, T* __restrict__ o_lat) {
  extern __shared__ float sm[];
  const int W = pages.width, WS = W | 1;   // odd stride: lanes read a column of keys without bank conflicts
  float* sk = sm;                          // [kLaK][WS]
  float* sq = sk + kLaK * WS;              // [kLaQ][W]
  float* so = sq + kLaQ * W;               // [kLaQ][R]
  float* sp = so + kLaQ * R;               // [kLaQ][kLaK]
  const int h = blockIdx.y, split = blockIdx.z, S = gridDim.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // tile -> (sequence, first query)
  int tile = blockIdx.x, b = 0, n0 = -1, cnt = 0;
  for (; b < sb.n_seq; ++b) {
    const int len = sb.cu[b + 1] - sb.cu[b], tiles = (len + kLaQ - 1) / kLaQ;
    if (tile < tiles) {
      n0 = sb.cu[b] + tile * kLaQ;
      cnt = min(kLaQ, len - tile * kLaQ);
      break;
    }
    tile -= tiles;
  }
  if (n0 < 0) return;
  const int slot = sb.ids[b];
  const int pos0 = sb.start[b] + n0 - sb.cu[b];
  const int n_keys = pos0 + cnt;
  const int tiles_k = (n_keys + kLaK - 1) / kLaK, per = (tiles_k + S - 1) / S;
  const int kt0 = split * per, kt1 = min(tiles_k, kt0 + per);
  for (int i = threadIdx.x; i < kLaQ * W; i += blockDim.x) {
    const int q = i / W;
    sq[i] = q < cnt ? ldf(qf + (static_cast<int64_t>(n0 + q) * H + h) * W + i % W) : 0.f;
  }
  for (int i = threadIdx.x; i < kLaQ * R; i += blockDim.x) so[i] = 0.f;
  constexpr int kMine = kLaQ / kLaWarps;
  float m[kMine], l[kMine];
#pragma unroll
  for (int j = 0; j < kMine; ++j) { m[j] = -INFINITY; l[j] = 0.f; }
  for (int kt = kt0; kt < kt1; ++kt) {
    __syncthreads();
    for (int k = warp; k < kLaK; k += kLaWarps) {
      const int pos = kt * kLaK + k;
      const int64_t row = pos < n_keys ? page_row(pages, slot, pos) : -1;
      const T* src = static_cast<const T*>(pages.pool) + (row < 0 ? 0 : row) * W;
      for (int i = lane; i < W; i += 32) sk[k * WS + i] = row < 0 ? 0.f : ldf(src + i);
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < kMine; ++j) {
      const int q = warp + j * kLaWarps;
      if (q >= cnt) continue;   // warp-uniform
      float s = 0.f;
      const float* qv = sq + q * W;
      const float* kv = sk + lane * WS;
#pragma unroll 4
      for (int i = 0; i < W; ++i) s = fmaf(qv[i], kv[i], s);
      s = (kt * kLaK + lane <= pos0 + q) ? s * scale : -INFINITY;
      const float mn = fmaxf(m[j], warp_max(s));
      if (mn == -INFINITY) {
        sp[q * kLaK + lane] = 0.f;
        __syncwarp();
        continue;
      }
      const float p = expf(s - mn), a = expf(m[j] - mn);
      l[j] = l[j] * a + warp_sum(p);
      m[j] = mn;
      sp[q * kLaK + lane] = p;
      __syncwarp();
      for (int c = lane; c < R; c += 32) {
        float o = so[q * R + c] * a;
#pragma unroll 8
        for (int k = 0; k < kLaK; ++k) o = fmaf(sp[q * kLaK + k], sk[k * WS + c], o);
        so[q * R + c] = o;
      }
      __syncwarp();
    }
  }
#pragma unroll
  for (int j = 0; j < kMine; ++j) {
    const int q = warp + j * kLaWarps;
    if (q >= cnt) continue;
    const int64_t nh = static_cast<int64_t>(n0 + q) * H + h;
    if (S == 1) {
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

// ---- table-routed experts ---------------------------------------------------------------------------------------------
__device__ __forceinline__ float clamped_glu(float g, float u, const GluArgs& a) {
  g = fminf(g, a.limit);
  u = fminf(fmaxf(u, -a.limit), a.limit);
  return g * sigmoid_f(a.alpha * g) * (u + 1.f);
}

constexpr int kExpWarps = 8;

// h[m * top + j, i] = glu(gate_e[i] . x[m], up_e[i] . x[m]) with e = table[token m, j]; w_gate_up [E, 2 I, D].
template <typename T, bool kVec>
__global__ void __launch_bounds__(kExpWarps * 32)
table_experts_up_kernel(const T* __restrict__ x, const int* __restrict__ tokens, const int* __restrict__ table, int vocab,
                        int top, int E, const T* __restrict__ w, GluArgs glu, T* __restrict__ h, int D, int I, int* status) {
  const int pair = blockIdx.x, m = pair / top;
  const int tok = tokens[m];
  const int e = tok >= 0 && tok < vocab ? table[static_cast<int64_t>(tok) * top + pair % top] : -1;
  if (e < 0 || e >= E) {
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
#pragma unroll 2
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
    if (lane == 0) stf(h + static_cast<int64_t>(pair) * I + i, clamped_glu(g, u, glu));
  }
}

// x[m, d] += 1 / top * sum_j down_e(j)[d] . h[m * top + j]; w_down [E, D, I].
template <typename T, bool kVec>
__global__ void __launch_bounds__(kExpWarps * 32)
table_experts_down_kernel(const T* __restrict__ h, const int* __restrict__ tokens, const int* __restrict__ table, int vocab,
                          int top, int E, const T* __restrict__ w, float* __restrict__ x, int D, int I) {
  const int m = blockIdx.x;
  const int tok = tokens[m];
  if (tok < 0 || tok >= vocab) return;
  const int lane = threadIdx.x & 31;
  for (int d = blockIdx.y * kExpWarps + (threadIdx.x >> 5); d < D; d += gridDim.y * kExpWarps) {
    float acc = 0.f;
    for (int j = 0; j < top; ++j) {
      const int e = table[static_cast<int64_t>(tok) * top + j];
      if (e < 0 || e >= E) continue;
      const T* wr = w + (static_cast<int64_t>(e) * D + d) * I;
      const T* hr = h + (static_cast<int64_t>(m) * top + j) * I;
      if constexpr (kVec) {
        constexpr int V = Vec16<T>::n;
#pragma unroll 2
        for (int k = lane * V; k < I; k += 32 * V) {
          float hv[V], wv[V];
          Vec16<T>::load(hr + k, hv);
          Vec16<T>::load(wr + k, wv);
#pragma unroll
          for (int q = 0; q < V; ++q) acc = fmaf(hv[q], wv[q], acc);
        }
      } else {
        for (int k = lane; k < I; k += 32) acc = fmaf(ldf(hr + k), ldf(wr + k), acc);
      }
    }
    acc = warp_sum(acc);
    if (lane == 0) x[static_cast<int64_t>(m) * D + d] += acc / top;
  }
}

__global__ void moe_gather_rows_kernel(const __nv_bfloat16* __restrict__ x, const int* __restrict__ idx,
                                       const int* __restrict__ pos, const int* __restrict__ offs_end,
                                       const int* __restrict__ counts, int top, __nv_bfloat16* __restrict__ xs,
                                       int* __restrict__ row_of, int D) {
  const int p = blockIdx.x, e = idx[p];
  const int row = offs_end[e] - counts[e] + pos[p];
  if (threadIdx.x == 0) row_of[p] = row;
  const uint4* src = reinterpret_cast<const uint4*>(x + static_cast<int64_t>(p / top) * D);
  uint4* dst = reinterpret_cast<uint4*>(xs + static_cast<int64_t>(row) * D);
  for (int i = threadIdx.x; i < D / 8; i += blockDim.x) dst[i] = src[i];
}

__global__ void clamped_glu_kernel(const __nv_bfloat16* __restrict__ gu, GluArgs glu, __nv_bfloat16* __restrict__ h,
                                   int64_t n8, int I8) {
  for (int64_t i = blockIdx.x * static_cast<int64_t>(blockDim.x) + threadIdx.x; i < n8;
       i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t r = i / I8, c = i % I8;
    float g[8], u[8];
    Vec16<__nv_bfloat16>::load(gu + (r * 2 * I8 + c) * 8, g);
    Vec16<__nv_bfloat16>::load(gu + (r * 2 * I8 + I8 + c) * 8, u);
    uint32_t o[4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
      o[j] = pack_bf16x2(clamped_glu(g[2 * j], u[2 * j], glu), clamped_glu(g[2 * j + 1], u[2 * j + 1], glu));
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

// Opts a kernel into `bytes` of dynamic shared memory once per new maximum.
template <typename K>
cudaError_t want_smem(K kernel, int bytes, int& have) {
  if (bytes <= 48 * 1024 || bytes <= have) return cudaSuccess;
  if (bytes > 227 * 1024) return cudaErrorInvalidValue;
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e == cudaSuccess) have = bytes;
  return e;
}

template <typename T>
cudaError_t latent_attention_t(const SeqBatch& sb, const T* qf, const PagedRows& pages, int R, const float* sink, float scale,
                               int H, int n_splits, float* part_o, float* part_ml, T* o_lat, cudaStream_t st) {
  static int have = 0;
  const int smem = 4 * (kLaK * (pages.width + 1) + kLaQ * pages.width + kLaQ * R + kLaQ * kLaK);
  cudaError_t e = want_smem(latent_attn_kernel<T>, smem, have);
  if (e != cudaSuccess) return e;
  const dim3 grid(sb.n_tok / kLaQ + sb.n_seq, H, n_splits);
  latent_attn_kernel<T><<<grid, kLaWarps * 32, smem, st>>>(sb, qf, pages, R, sink, scale, H, part_o, part_ml, o_lat);
  if (n_splits > 1) latent_merge_kernel<T><<<sb.n_tok * H, 128, 0, st>>>(part_o, part_ml, sink, H, R, n_splits, o_lat);
  return cudaGetLastError();
}

template <typename T>
cudaError_t absorb_q_t(const SeqBatch& sb, const T* q, const T* w_uk, T* qf, int H, int dn, int dr, int R,
                       const RopeTable& rope, cudaStream_t st) {
  static int have = 0;
  const int smem = 4 * kAbsTok * (dn + dr);
  cudaError_t e = want_smem(mla_absorb_q_kernel<T>, smem, have);
  if (e != cudaSuccess) return e;
  const int tiles = (sb.n_tok + kAbsTok - 1) / kAbsTok;
  const int z = tiles * H < 296 ? min(4, (R + 127) / 128) : 1;
  mla_absorb_q_kernel<T><<<dim3(tiles, H, z), 128, smem, st>>>(sb, q, w_uk, qf, H, dn, dr, R, rope);
  return cudaGetLastError();
}

template <typename T>
cudaError_t absorb_out_t(const T* o_lat, const T* w_uv, T* o, int n_tok, int H, int dv, int R, cudaStream_t st) {
  static int have = 0;
  const int smem = 4 * kAbsTok * R;
  cudaError_t e = want_smem(mla_absorb_out_kernel<T>, smem, have);
  if (e != cudaSuccess) return e;
  const int tiles = (n_tok + kAbsTok - 1) / kAbsTok;
  const int z = tiles * H < 296 ? min(8, (dv + 7) / 8) : 1;
  mla_absorb_out_kernel<T><<<dim3(tiles, H, z), 256, smem, st>>>(o_lat, w_uv, o, n_tok, H, dv, R);
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
  if (f32_out) norm_rows_kernel<float><<<rows, threads_for(D), 0, st>>>(mode, x, gamma, beta, static_cast<float*>(out), D, eps);
  else norm_rows_kernel<__nv_bfloat16><<<rows, threads_for(D), 0, st>>>(mode, x, gamma, beta, static_cast<__nv_bfloat16*>(out), D, eps);
  return cudaGetLastError();
}

cudaError_t launch_rows_linear(bool f32, const void* x, int64_t ldx, const void* w, int64_t ldw, void* y, int64_t ldy,
                               int M, int N, int K, int act, int out_mode, cudaStream_t st) {
  if (M < 1 || N < 1 || K < 1) return cudaErrorInvalidValue;
  return f32 ? rows_linear_t<float>(x, ldx, w, ldw, y, ldy, M, N, K, act, out_mode, st)
             : rows_linear_t<__nv_bfloat16>(x, ldx, w, ldw, y, ldy, M, N, K, act, out_mode, st);
}

cudaError_t launch_mla_prepare(bool f32, const SeqBatch& sb, const void* y, int64_t ldy, int q_rank, int R, int dr,
                               const float* q_gamma, const float* kv_gamma, float eps, const RopeTable& rope,
                               const PagedRows& pages, void* cq, void* lat, int* status, cudaStream_t st) {
  const int th = threads_for(q_rank + R + dr);
  if (f32)
    mla_prepare_kernel<float><<<sb.n_tok, th, 0, st>>>(sb, static_cast<const float*>(y), ldy, q_rank, R, dr, q_gamma, kv_gamma,
                                                       eps, rope, pages, static_cast<float*>(cq), static_cast<float*>(lat), status);
  else
    mla_prepare_kernel<__nv_bfloat16><<<sb.n_tok, th, 0, st>>>(sb, static_cast<const __nv_bfloat16*>(y), ldy, q_rank, R, dr, q_gamma,
                                                               kv_gamma, eps, rope, pages, static_cast<__nv_bfloat16*>(cq),
                                                               static_cast<__nv_bfloat16*>(lat), status);
  return cudaGetLastError();
}

cudaError_t launch_mla_rope_qk(bool f32, const SeqBatch& sb, void* q, const void* kn, int64_t ldkn, const void* lat,
                               int64_t ldlat, int R, void* k, int H, int dn, int dr, const RopeTable& rope, cudaStream_t st) {
  if (f32)
    mla_rope_qk_kernel<float><<<sb.n_tok, 256, 0, st>>>(sb, static_cast<float*>(q), static_cast<const float*>(kn), ldkn,
                                                        static_cast<const float*>(lat), ldlat, R, static_cast<float*>(k), H, dn, dr, rope);
  else
    mla_rope_qk_kernel<__nv_bfloat16><<<sb.n_tok, 256, 0, st>>>(
        sb, static_cast<__nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(kn), ldkn, static_cast<const __nv_bfloat16*>(lat),
        ldlat, R, static_cast<__nv_bfloat16*>(k), H, dn, dr, rope);
  return cudaGetLastError();
}

cudaError_t launch_mla_absorb_q(bool f32, const SeqBatch& sb, const void* q, const void* w_uk, void* qf, int H, int dn,
                                int dr, int R, const RopeTable& rope, cudaStream_t st) {
  return f32 ? absorb_q_t<float>(sb, static_cast<const float*>(q), static_cast<const float*>(w_uk), static_cast<float*>(qf), H, dn,
                                 dr, R, rope, st)
             : absorb_q_t<__nv_bfloat16>(sb, static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(w_uk),
                                         static_cast<__nv_bfloat16*>(qf), H, dn, dr, R, rope, st);
}

cudaError_t launch_mla_absorb_out(bool f32, const void* o_lat, const void* w_uv, void* o, int n_tok, int H, int dv, int R,
                                  cudaStream_t st) {
  return f32 ? absorb_out_t<float>(static_cast<const float*>(o_lat), static_cast<const float*>(w_uv), static_cast<float*>(o), n_tok,
                                   H, dv, R, st)
             : absorb_out_t<__nv_bfloat16>(static_cast<const __nv_bfloat16*>(o_lat), static_cast<const __nv_bfloat16*>(w_uv),
                                           static_cast<__nv_bfloat16*>(o), n_tok, H, dv, R, st);
}

cudaError_t launch_latent_attention(bool f32, const SeqBatch& sb, const void* qf, const PagedRows& pages, int R,
                                    const float* sink, float scale, int H, int n_splits, float* part_o, float* part_ml,
                                    void* o_lat, cudaStream_t st) {
  if (n_splits < 1 || (n_splits > 1 && (part_o == nullptr || part_ml == nullptr))) return cudaErrorInvalidValue;
  return f32 ? latent_attention_t<float>(sb, static_cast<const float*>(qf), pages, R, sink, scale, H, n_splits, part_o, part_ml,
                                         static_cast<float*>(o_lat), st)
             : latent_attention_t<__nv_bfloat16>(sb, static_cast<const __nv_bfloat16*>(qf), pages, R, sink, scale, H, n_splits,
                                                 part_o, part_ml, static_cast<__nv_bfloat16*>(o_lat), st);
}

cudaError_t launch_table_experts_up(bool f32, const void* x, const int* tokens, const int* table, int vocab, int top, int E,
                                    const void* w, GluArgs glu, void* h, int M, int D, int I, int* status, cudaStream_t st) {
  const int per = (I + kExpWarps - 1) / kExpWarps;
  const dim3 grid(M * top, per < 64 ? per : 64);
  const bool vec = D % (f32 ? 4 : 8) == 0;
#define B200_UP(T, V)                                                                                                      \
  table_experts_up_kernel<T, V><<<grid, kExpWarps * 32, 0, st>>>(static_cast<const T*>(x), tokens, table, vocab, top, E,    \
                                                                 static_cast<const T*>(w), glu, static_cast<T*>(h), D, I, status)
  if (f32) { if (vec) B200_UP(float, true); else B200_UP(float, false); }
  else { if (vec) B200_UP(__nv_bfloat16, true); else B200_UP(__nv_bfloat16, false); }
#undef B200_UP
  return cudaGetLastError();
}

cudaError_t launch_table_experts_down(bool f32, const void* h, const int* tokens, const int* table, int vocab, int top,
                                      int E, const void* w, float* x, int M, int D, int I, cudaStream_t st) {
  const int per = (D + kExpWarps - 1) / kExpWarps;
  const dim3 grid(M, per < 256 ? per : 256);
  const bool vec = I % (f32 ? 4 : 8) == 0;
#define B200_DN(T, V)                                                                                                      \
  table_experts_down_kernel<T, V><<<grid, kExpWarps * 32, 0, st>>>(static_cast<const T*>(h), tokens, table, vocab, top, E,  \
                                                                   static_cast<const T*>(w), x, D, I)
  if (f32) { if (vec) B200_DN(float, true); else B200_DN(float, false); }
  else { if (vec) B200_DN(__nv_bfloat16, true); else B200_DN(__nv_bfloat16, false); }
#undef B200_DN
  return cudaGetLastError();
}

cudaError_t launch_moe_gather_rows(const __nv_bfloat16* x, const int* idx, const int* pos, const int* offs_end,
                                   const int* counts, int top, __nv_bfloat16* xs, int* row_of, int M, int D, cudaStream_t st) {
  if (D % 8 != 0) return cudaErrorInvalidValue;
  moe_gather_rows_kernel<<<M * top, 128, 0, st>>>(x, idx, pos, offs_end, counts, top, xs, row_of, D);
  return cudaGetLastError();
}
cudaError_t launch_clamped_glu(const __nv_bfloat16* gu, GluArgs glu, __nv_bfloat16* h, int rows, int I, cudaStream_t st) {
  if (I % 8 != 0) return cudaErrorInvalidValue;
  const int64_t n8 = static_cast<int64_t>(rows) * (I / 8);
  const int grid = static_cast<int>((n8 + 255) / 256 < 148 * 16 ? (n8 + 255) / 256 : 148 * 16);
  clamped_glu_kernel<<<grid > 0 ? grid : 1, 256, 0, st>>>(gu, glu, h, n8, I / 8);
  return cudaGetLastError();
}
cudaError_t launch_moe_combine_rows(const __nv_bfloat16* ys, const int* row_of, int top, float w, float* x, int M, int D,
                                    cudaStream_t st) {
  if (D % 8 != 0) return cudaErrorInvalidValue;
  moe_combine_rows_kernel<<<M, 128, 0, st>>>(ys, row_of, top, w, x, D);
  return cudaGetLastError();
}

}  // namespace b200
