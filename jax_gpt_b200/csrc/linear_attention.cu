// Linear-attention layers with a matrix state per head on packed batches (any sizes, fp32 or bf16 activations):
//
//   S_t = a_t S_(t-1) + b_t k_t v_t^T        o_t = q_scale S_t^T q_t
//
// with a fixed decay per head (a_t = decay, b_t = 1), with a decay per key channel (a_t = diag(alpha_t), b_t = 1, log alpha =
// log sigmoid(w2 low + bias2) / tau; Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training"), or
// with exponential gates from log values i, f and a running maximum
// m (Beck et al., "xLSTM: Extended Long Short-Term Memory"):
//   m_t = max(f_t + m_(t-1), i_t), a_t = exp(f_t + m_(t-1) - m_t), b_t = exp(i_t - m_t), n_t = a_t n_(t-1) + b_t k_t,
//   o_t / (max(|q_scale n_t . q_t|, exp(-m_t)) + den_eps)
// i = cap tanh(raw / cap), f = log sigmoid(cap tanh(raw / cap)).
//
// The gated scans leave the numerators in y and {n . q in two parts, exp(-m)} in `den`; head_norm_gate divides, applies the
// RMS norm over equal pieces of the row, the gain and the output gate. The chunked tensor-core form is in
// ssd_scan_sm100.cu. All gates, states and norms are fp32. This file is built without fast-math.
#include "serve_common.cuh"
#include "serve_kernels.cuh"

namespace b200 {

namespace {

__device__ __forceinline__ float soft_cap(float x, float cap) { return cap * tanhf(x / cap); }

// log input and forget gate of (row, head)
__device__ __forceinline__ void log_gates(const LinGates& g, int64_t row, int h, int H, float& i, float& f) {
  const float* p = g.raw + row * g.ld;
  i = soft_cap(p[h] + g.bias[h], g.cap);
  f = -softplus_f(-soft_cap(p[H + h] + g.bias[H + h], g.cap));
}

// decay of (row, head, key channel), less 1: S + (decay - 1) S keeps the distance of slow decays from 1
template <typename T>
__device__ __forceinline__ float channel_decay(const LinGates& g, int64_t row, int hn) {
  const T *x = static_cast<const T*>(g.low) + row * g.ld_low, *w = static_cast<const T*>(g.w2) + static_cast<int64_t>(hn) * g.R;
  float z = g.bias2[hn];
  for (int r = 0; r < g.R; ++r) z = fmaf(ldf(x + r), ldf(w + r), z);
  return expm1f(-softplus_f(-z) * g.inv_tau);
}

enum LinKind : int { kFixed = 0, kGatedExp = 1, kChannel = 2 };

template <typename T>
__device__ __forceinline__ float qkv_at(const T* p, int silu) {
  const float v = ldf(p);
  return silu ? rnd<T>(silu_f(v)) : v;
}

// ---- token by token ----------------------------------------------------------------------------------------------------
// Block: one head of one sequence, 16 columns of the state; thread (p, g) holds rows g, g + 8, ... of column p. The blocks
// of the first columns also carry n and m (kGated).
constexpr int kScanP = 16, kScanG = 8, kScanTok = 16;

template <typename T, int NS, int kKind>
__global__ void __launch_bounds__(kScanP * kScanG)
linear_scan_kernel(const SeqBatch sb, const T* __restrict__ qkv, int64_t ld, const LinGates gates, float* __restrict__ state,
                   float* __restrict__ y, const LinShape s) {
  constexpr bool kGated = kKind == kGatedExp;
  extern __shared__ float sm[];
  const int N = s.N, P = s.P;
  float* sK = sm;                       // [kScanTok][N]
  float* sQ = sK + kScanTok * N;        // [kScanTok][N]
  float* sV = sQ + kScanTok * N;        // [kScanTok][kScanP]
  float* sA = sV + kScanTok * kScanP;   // [kScanTok] state factor
  float* sB = sA + kScanTok;            // [kScanTok] input factor
  float* sE = sB + kScanTok;            // [kScanTok] exp(-m)
  float* sC = sE + kScanTok;            // [kScanTok][N] decays of the key channels (kChannel)
  const int h = blockIdx.x, p0 = blockIdx.y * kScanP, b = blockIdx.z;
  const int g = threadIdx.x % kScanG, p = threadIdx.x / kScanG;   // the eight row groups of a column are neighbours
  const int first = sb.cu[b], len = sb.cu[b + 1] - first;
  const int inner = s.H * P;
  const bool fresh = sb.start[b] == 0, live = p0 + p < P, own = kGated && blockIdx.y == 0;
  float* st = state + (static_cast<int64_t>(sb.ids[b]) * s.H + h) * N * P;
  const float* vec = kGated ? gates.vec + (static_cast<int64_t>(sb.ids[b]) * s.H + h) * (N + 1) : nullptr;
  float S[NS], nn[kGated ? NS : 1];
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = g + i * kScanG;
    S[i] = (!fresh && live && n < N) ? st[static_cast<int64_t>(n) * P + p0 + p] : 0.f;
    if constexpr (kGated) nn[i] = (!fresh && n < N) ? vec[n] : 0.f;
  }
  float m = kGated && !fresh ? vec[N] : 0.f;   // thread 0's copy advances
  const float decay = kKind == kFixed ? gates.decay[h] : 0.f;
  for (int t0 = 0; t0 < len; t0 += kScanTok) {
    const int cnt = min(kScanTok, len - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < cnt * N; i += blockDim.x) {
      const T* row = qkv + static_cast<int64_t>(first + t0 + i / N) * ld + h * N + i % N;
      sQ[i] = qkv_at(row, s.silu);
      sK[i] = qkv_at(row + s.H * N, s.silu);
      if constexpr (kKind == kChannel) sC[i] = channel_decay<T>(gates, first + t0 + i / N, h * N + i % N);
    }
    for (int i = threadIdx.x; i < cnt * kScanP; i += blockDim.x)
      sV[i] = p0 + i % kScanP < P ? qkv_at(qkv + static_cast<int64_t>(first + t0 + i / kScanP) * ld + 2 * s.H * N + h * P + p0 + i % kScanP, s.silu) : 0.f;
    if constexpr (kGated) {
      if (threadIdx.x < cnt) {
        float li, lf;
        log_gates(gates, first + t0 + threadIdx.x, h, s.H, li, lf);
        sA[threadIdx.x] = lf;
        sB[threadIdx.x] = li;
      }
      __syncthreads();
      if (threadIdx.x == 0) {
        for (int t = 0; t < cnt; ++t) {
          const float lf = sA[t], li = sB[t], mn = fmaxf(lf + m, li);
          sA[t] = expf(lf + m - mn);
          sB[t] = expf(li - mn);
          sE[t] = expf(-mn);
          m = mn;
        }
      }
    }
    __syncthreads();
    for (int t = 0; t < cnt; ++t) {
      const float a = kGated ? sA[t] : decay, w = kGated ? sB[t] : 1.f, x = sV[t * kScanP + p] * w;
      float acc = 0.f, dot = 0.f;
#pragma unroll
      for (int i = 0; i < NS; ++i) {
        const int n = g + i * kScanG;
        if (n < N) {
          if constexpr (kKind == kChannel) S[i] += fmaf(S[i], sC[t * N + n], x * sK[t * N + n]);
          else S[i] = fmaf(S[i], a, x * sK[t * N + n]);
          acc = fmaf(S[i], sQ[t * N + n], acc);
          if constexpr (kGated) {
            nn[i] = fmaf(nn[i], a, w * sK[t * N + n]);
            dot = fmaf(nn[i], sQ[t * N + n], dot);
          }
        }
      }
#pragma unroll
      for (int o = 1; o < kScanG; o <<= 1) {
        acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if constexpr (kGated) dot += __shfl_xor_sync(0xffffffffu, dot, o);
      }
      const int64_t row = first + t0 + t;
      if (g == 0 && live) y[row * inner + h * P + p0 + p] = acc * s.q_scale;
      if (own && threadIdx.x == 0)
        *reinterpret_cast<float4*>(gates.den + (row * s.H + h) * 4) = make_float4(dot * s.q_scale, 0.f, sE[t], 0.f);
    }
  }
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = g + i * kScanG;
    if (live && n < N) st[static_cast<int64_t>(n) * P + p0 + p] = S[i];
  }
  if constexpr (kGated) {
    if (own && p == 0) {   // other blocks of the head may still read the slot's old values: head_norm_gate moves these there
      float* vn = gates.vec_new + (static_cast<int64_t>(b) * s.H + h) * (N + 1);
#pragma unroll
      for (int i = 0; i < NS; ++i) {
        const int n = g + i * kScanG;
        if (n < N) vn[n] = nn[i];
      }
      if (threadIdx.x == 0) vn[N] = m;
    }
  }
}

template <typename T, int kKind>
cudaError_t linear_scan_t(const SeqBatch& sb, const T* qkv, int64_t ld, const LinGates& g, float* state, float* y,
                          const LinShape& s, cudaStream_t st) {
  const dim3 grid(s.H, (s.P + kScanP - 1) / kScanP, sb.n_seq);
  const int smem = 4 * ((kKind == kChannel ? 3 : 2) * kScanTok * s.N + kScanTok * kScanP + 3 * kScanTok);
#define B200_SCAN(NS)                                                                                                 \
  {                                                                                                                   \
    static int have = 0;                                                                                              \
    const cudaError_t e = want_smem(linear_scan_kernel<T, NS, kKind>, smem, have);                                   \
    if (e != cudaSuccess) return e;                                                                                   \
    linear_scan_kernel<T, NS, kKind><<<grid, kScanP * kScanG, smem, st>>>(sb, qkv, ld, g, state, y, s);              \
  }
  if (s.N <= 64) B200_SCAN(8)
  else if (s.N <= 128) B200_SCAN(16)
  else if (s.N <= 256) B200_SCAN(32)
  else if (s.N <= 512) B200_SCAN(64)
  else return cudaErrorInvalidValue;
#undef B200_SCAN
  return cudaGetLastError();
}

// ---- one token -----------------------------------------------------------------------------------------------------------
// Block: up to 64 columns of one head of one sequence; thread (row r, column lane) streams V columns of every `rows`-th
// state row. The block of the first columns advances n and m.
constexpr int kStepThreads = 256, kStepCols = 64;

template <typename T, int V, int kKind>
__global__ void __launch_bounds__(kStepThreads)
linear_step_kernel(const SeqBatch sb, const T* __restrict__ qkv, int64_t ld, const LinGates gates, float* __restrict__ state,
                   float* __restrict__ y, const LinShape s) {
  constexpr bool kGated = kKind == kGatedExp;
  extern __shared__ float sm[];
  __shared__ float red[33];
  const int N = s.N, P = s.P;
  const int h = blockIdx.x, p0 = blockIdx.y * kStepCols, b = blockIdx.z, cols = min(kStepCols, P - p0);
  float* sq = sm;                 // [N]
  float* sk = sq + N;             // [N]
  float* sv = sk + N;             // [kStepCols]
  float* sc = sv + kStepCols;     // [N] decays of the key channels (kChannel)
  float* part = kKind == kChannel ? sc + N : sc;   // [rows][cols]
  const int slot = sb.ids[b];
  const bool fresh = sb.start[b] == 0;
  const int64_t row = sb.cu[b];
  const T* x = qkv + row * ld;
  constexpr int kLanes = kStepCols / V, kRows = kStepThreads / kLanes;
  constexpr int kAhead = V == 4 ? 8 : 16;   // state rows of a thread in flight; the first ones load before the gates are known
  const int r = threadIdx.x / kLanes, c = (threadIdx.x % kLanes) * V;
  const bool live = c < cols;
  float* st = state + (static_cast<int64_t>(slot) * s.H + h) * N * P + p0 + c;
  float S[kAhead][V];
  auto load = [&](int n0) {
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      const int n = n0 + i * kRows;
#pragma unroll
      for (int j = 0; j < V; ++j) S[i][j] = 0.f;
      if (live && !fresh && n < N) {
        const float* sp = st + static_cast<int64_t>(n) * P;
        if constexpr (V == 4) {
          const float4 f = *reinterpret_cast<const float4*>(sp);
          S[i][0] = f.x; S[i][1] = f.y; S[i][2] = f.z; S[i][3] = f.w;
        } else {
          S[i][0] = sp[0];
        }
      }
    }
  };
  load(r);
  for (int i = threadIdx.x; i < N; i += blockDim.x) {
    sq[i] = qkv_at(x + h * N + i, s.silu);
    sk[i] = qkv_at(x + (s.H + h) * N + i, s.silu);
    if constexpr (kKind == kChannel) sc[i] = channel_decay<T>(gates, row, h * N + i);
  }
  for (int i = threadIdx.x; i < cols; i += blockDim.x) sv[i] = qkv_at(x + 2 * s.H * N + h * P + p0 + i, s.silu);
  float a = 0.f, w = 1.f, m = 0.f;
  const float* vec = nullptr;
  if constexpr (kGated) {
    vec = gates.vec + (static_cast<int64_t>(slot) * s.H + h) * (N + 1);
    float li, lf;
    log_gates(gates, row, h, s.H, li, lf);
    const float m0 = fresh ? 0.f : vec[N];
    m = fmaxf(lf + m0, li);
    a = expf(lf + m0 - m);
    w = expf(li - m);
  } else if constexpr (kKind == kFixed) {
    a = gates.decay[h];
  }
  __syncthreads();
  if (live) {
    float acc[V], dx[V];
#pragma unroll
    for (int j = 0; j < V; ++j) { acc[j] = 0.f; dx[j] = w * sv[c + j]; }
    for (int n0 = r; n0 < N; n0 += kAhead * kRows) {
      if (n0 != r) load(n0);
#pragma unroll
      for (int i = 0; i < kAhead; ++i) {
        const int n = n0 + i * kRows;
        if (n >= N) break;
        float* sp = st + static_cast<int64_t>(n) * P;
        const float kn = sk[n], qn = sq[n], an = kKind == kChannel ? sc[n] : a;
#pragma unroll
        for (int j = 0; j < V; ++j) {
          if constexpr (kKind == kChannel) S[i][j] += fmaf(S[i][j], an, dx[j] * kn);
          else S[i][j] = fmaf(S[i][j], an, dx[j] * kn);
          acc[j] = fmaf(S[i][j], qn, acc[j]);
        }
        if constexpr (V == 4) *reinterpret_cast<float4*>(sp) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
        else sp[0] = S[i][0];
      }
    }
#pragma unroll
    for (int j = 0; j < V; ++j) part[r * kStepCols + c + j] = acc[j];
  }
  if constexpr (kGated) {
    if (blockIdx.y == 0) {
      float dot = 0.f;
      float* vn = gates.vec_new + (static_cast<int64_t>(b) * s.H + h) * (N + 1);
      for (int n = threadIdx.x; n < N; n += blockDim.x) {
        const float v = fmaf(fresh ? 0.f : vec[n], a, w * sk[n]);
        vn[n] = v;
        dot = fmaf(v, sq[n], dot);
      }
      dot = block_sum(dot, red);
      if (threadIdx.x == 0) {
        vn[N] = m;
        *reinterpret_cast<float4*>(gates.den + (row * s.H + h) * 4) = make_float4(dot * s.q_scale, 0.f, expf(-m), 0.f);
      }
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < cols; i += blockDim.x) {
    float v = 0.f;
#pragma unroll
    for (int q = 0; q < kRows; ++q) v += part[q * kStepCols + i];
    y[row * s.H * P + h * P + p0 + i] = v * s.q_scale;
  }
}

template <typename T, int kKind>
cudaError_t linear_step_t(const SeqBatch& sb, const T* qkv, int64_t ld, const LinGates& g, float* state, float* y,
                          const LinShape& s, cudaStream_t st) {
  const dim3 grid(s.H, (s.P + kStepCols - 1) / kStepCols, sb.n_seq);
  if (s.P % 4 == 0) {
    static int have = 0;
    const int smem = 4 * ((kKind == kChannel ? 3 : 2) * s.N + kStepCols + kStepThreads * 4);
    const cudaError_t e = want_smem(linear_step_kernel<T, 4, kKind>, smem, have);
    if (e != cudaSuccess) return e;
    linear_step_kernel<T, 4, kKind><<<grid, kStepThreads, smem, st>>>(sb, qkv, ld, g, state, y, s);
  } else {
    static int have = 0;
    const int smem = 4 * ((kKind == kChannel ? 3 : 2) * s.N + kStepCols + kStepThreads);
    const cudaError_t e = want_smem(linear_step_kernel<T, 1, kKind>, smem, have);
    if (e != cudaSuccess) return e;
    linear_step_kernel<T, 1, kKind><<<grid, kStepThreads, smem, st>>>(sb, qkv, ld, g, state, y, s);
  }
  return cudaGetLastError();
}

// ---- normalisation, gain, output gate --------------------------------------------------------------------------------
// 1 / (max(|n . q|, exp(-m)) + den_eps) of (row, piece); pieces are the heads
__device__ __forceinline__ float inv_den(const HeadNorm& a, int64_t piece) {
  if (a.den == nullptr) return 1.f;
  const float4 d = *reinterpret_cast<const float4*>(a.den + piece * 4);
  return 1.f / (fmaxf(fabsf(d.x + d.y), d.z) + a.den_eps);
}

// The last row of a sequence takes the advanced n and m of its head to the sequence's slot.
__device__ __forceinline__ void commit_vec(const HeadNorm& a, const SeqBatch& sb, int n, int h, int tid, int threads) {
  if (a.vec == nullptr) return;
  const int b = sb.tok_seq[n];
  if (n != sb.cu[b + 1] - 1) return;
  const float* src = a.vec_new + (static_cast<int64_t>(b) * a.parts + h) * a.vec_len;
  float* dst = a.vec + (static_cast<int64_t>(sb.ids[b]) * a.parts + h) * a.vec_len;
#pragma unroll 8
  for (int i = tid; i < a.vec_len; i += threads) dst[i] = src[i];
}

template <typename TY, typename T>
__global__ void head_norm_gate_kernel(const SeqBatch sb, const TY* __restrict__ y, const T* __restrict__ z, int64_t ldz,
                                      const float* __restrict__ gamma, T* __restrict__ out, int D, const HeadNorm a) {
  extern __shared__ float buf[];   // [part]
  __shared__ float red[33];
  const int n = blockIdx.x, h = blockIdx.y, part = D / a.parts, c0 = h * part;
  const float w = inv_den(a, static_cast<int64_t>(n) * a.parts + h);
  float ss = 0.f;
  for (int i = threadIdx.x; i < part; i += blockDim.x) {
    const float v = ldf(y + static_cast<int64_t>(n) * D + c0 + i) * w;
    buf[i] = v;
    ss += v * v;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / part + a.eps);
  for (int i = threadIdx.x; i < part; i += blockDim.x) {
    const float zv = ldf(z + static_cast<int64_t>(n) * ldz + c0 + i);
    stf(out + static_cast<int64_t>(n) * D + c0 + i, buf[i] * inv * gamma[c0 + i] * sigmoid_f(zv) * (a.gate == 1 ? zv : 1.f));
  }
  commit_vec(a, sb, n, h, threadIdx.x, blockDim.x);
}

template <typename TY>
__device__ __forceinline__ void ld8(const TY* p, float (&f)[8]) {
  if constexpr (sizeof(TY) == 2) {
    Vec16<TY>::load(p, f);
  } else {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
}

// Eight features per thread and step; kThr threads own one piece of one row. bf16 out, part <= 8 * kThr * kIt.
template <typename TY, int kIt, int kThr>
__global__ void __launch_bounds__(256)
head_norm_gate_vec_kernel(const SeqBatch sb, const TY* __restrict__ y, const __nv_bfloat16* __restrict__ z, int64_t ldz,
                          const float* __restrict__ gamma, __nv_bfloat16* __restrict__ out, int pieces, int D, const HeadNorm a) {
  __shared__ float red[33];
  const int piece = blockIdx.x * (256 / kThr) + threadIdx.x / kThr, tid = threadIdx.x % kThr;
  const bool live = kThr == 256 || piece < pieces;   // every lane takes part in the shuffles
  const int n = live ? piece / a.parts : 0, h = live ? piece % a.parts : 0, part = D / a.parts, c0 = h * part;
  const float w = inv_den(a, live ? piece : 0);
  float v[kIt][8], zv[kIt][8];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + tid) * 8;
    if (live && i < part) {
      ld8(y + static_cast<int64_t>(n) * D + c0 + i, v[k]);
      Vec16<__nv_bfloat16>::load(z + static_cast<int64_t>(n) * ldz + c0 + i, zv[k]);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        v[k][j] *= w;
        ss += v[k][j] * v[k][j];
      }
    }
  }
  if constexpr (kThr == 256) {
    ss = block_sum(ss, red);
  } else {
#pragma unroll
    for (int o = kThr / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  }
  if (!live) return;
  const float inv = 1.f / sqrtf(ss / part + a.eps);
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + tid) * 8;
    if (i < part) {
      float g[8];
      ld8(gamma + c0 + i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) g[j] *= v[k][j] * inv * __fdividef(a.gate == 1 ? zv[k][j] : 1.f, 1.f + __expf(-zv[k][j]));
      *reinterpret_cast<uint4*>(out + static_cast<int64_t>(n) * D + c0 + i) =
          make_uint4(pack_bf16x2(g[0], g[1]), pack_bf16x2(g[2], g[3]), pack_bf16x2(g[4], g[5]), pack_bf16x2(g[6], g[7]));
    }
  }
  commit_vec(a, sb, n, h, tid, kThr);
}

template <typename TY, typename T>
cudaError_t head_norm_gate_t(const SeqBatch& sb, const TY* y, const T* z, int64_t ldz, const float* gamma, T* out, int D,
                             const HeadNorm& a, cudaStream_t st) {
  const int part = D / a.parts;
  if constexpr (sizeof(T) == 2) {
    if (part % 8 == 0 && ldz % 8 == 0 && part <= 16384 &&
        ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(gamma) |
          reinterpret_cast<uintptr_t>(out)) & 15) == 0) {
      const int pieces = sb.n_tok * a.parts;
#define B200_HN(IT, THR) \
  head_norm_gate_vec_kernel<TY, IT, THR><<<(pieces + 256 / THR - 1) / (256 / THR), 256, 0, st>>>(sb, y, z, ldz, gamma, out, pieces, D, a)
      if (part <= 64) B200_HN(1, 8);
      else if (part <= 128) B200_HN(1, 16);
      else if (part <= 256) B200_HN(1, 32);
      else if (part <= 512) B200_HN(2, 32);
      else if (part <= 2048) B200_HN(1, 256);
      else if (part <= 4096) B200_HN(2, 256);
      else if (part <= 8192) B200_HN(4, 256);
      else B200_HN(8, 256);
#undef B200_HN
      return cudaGetLastError();
    }
  }
  static int have = 0;
  const cudaError_t e = want_smem(head_norm_gate_kernel<TY, T>, part * 4, have);
  if (e != cudaSuccess) return e;
  const int th = part >= 1024 ? 256 : (part >= 256 ? 128 : 64);
  head_norm_gate_kernel<TY, T><<<dim3(sb.n_tok, a.parts), th, part * 4, st>>>(sb, y, z, ldz, gamma, out, D, a);
  return cudaGetLastError();
}

}  // namespace

#define B200_LIN(FN)                                                                                                    \
  {                                                                                                                     \
    if (f32) {                                                                                                          \
      const float* x = static_cast<const float*>(qkv);                                                                  \
      if (g.low != nullptr) return FN<float, kChannel>(sb, x, ld, g, state, y, s, st);                                  \
      return g.raw != nullptr ? FN<float, kGatedExp>(sb, x, ld, g, state, y, s, st) : FN<float, kFixed>(sb, x, ld, g, state, y, s, st); \
    }                                                                                                                   \
    const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(qkv);                                                    \
    if (g.low != nullptr) return FN<__nv_bfloat16, kChannel>(sb, x, ld, g, state, y, s, st);                            \
    return g.raw != nullptr ? FN<__nv_bfloat16, kGatedExp>(sb, x, ld, g, state, y, s, st)                               \
                            : FN<__nv_bfloat16, kFixed>(sb, x, ld, g, state, y, s, st);                                 \
  }
cudaError_t launch_linear_scan(bool f32, const SeqBatch& sb, const void* qkv, int64_t ld, const LinGates& g, float* state, float* y,
                               const LinShape& s, cudaStream_t st) {
  B200_LIN(linear_scan_t)
}

cudaError_t launch_linear_step(bool f32, const SeqBatch& sb, const void* qkv, int64_t ld, const LinGates& g, float* state, float* y,
                               const LinShape& s, cudaStream_t st) {
  B200_LIN(linear_step_t)
}
#undef B200_LIN

cudaError_t launch_head_norm_gate(bool f32, bool y_f32, const SeqBatch& sb, const void* y, const void* z, int64_t ldz,
                                  const float* gamma, void* out, int D, const HeadNorm& a, cudaStream_t st) {
  if (a.parts < 1 || D % a.parts != 0) return cudaErrorInvalidValue;
  if (f32)
    return head_norm_gate_t<float, float>(sb, static_cast<const float*>(y), static_cast<const float*>(z), ldz, gamma,
                                          static_cast<float*>(out), D, a, st);
  const __nv_bfloat16* zb = static_cast<const __nv_bfloat16*>(z);
  __nv_bfloat16* o = static_cast<__nv_bfloat16*>(out);
  return y_f32 ? head_norm_gate_t<float, __nv_bfloat16>(sb, static_cast<const float*>(y), zb, ldz, gamma, o, D, a, st)
               : head_norm_gate_t<__nv_bfloat16, __nv_bfloat16>(sb, static_cast<const __nv_bfloat16*>(y), zb, ldz, gamma, o, D, a, st);
}

}  // namespace b200
