// State-space (Mamba-2) layers on packed batches: causal depthwise convolution with a ring of past inputs, the
// recurrence token by token with the state in registers (any sizes, fp32 or bf16 activations), the one-launch decode
// step and the gated RMS norm over groups. The chunked tensor-core form of the recurrence is in ssd_scan_sm100.cu.
//
//   S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T        y_t = S_t^T C_t + D x_t
//
// Step sizes, decays and states are fp32 throughout. This file is built without fast-math.
#include "serve_kernels.cuh"

#include "serve_common.cuh"

namespace b200 {

namespace {

// ---- convolution -----------------------------------------------------------------------------------------------------
template <typename T>
__global__ void ssm_conv_kernel(const SeqBatch sb, const T* __restrict__ x, int64_t ldx, const float* __restrict__ w,
                                const float* __restrict__ bias, const float* __restrict__ ring, T* __restrict__ y, int C,
                                int taps) {
  const int n = blockIdx.x;
  const int b = sb.tok_seq[n], first = sb.cu[b], start = sb.start[b];
  const int pos = start + n - first;
  const float* rg = ring + static_cast<int64_t>(sb.ids[b]) * taps * C;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
    float acc = bias[c];
    for (int k = 0; k < taps; ++k) {
      const int p = pos - (taps - 1) + k;
      if (p < 0) continue;
      const float v = p >= start ? ldf(x + static_cast<int64_t>(first + p - start) * ldx + c) : rg[static_cast<int64_t>(p % taps) * C + c];
      acc = fmaf(w[static_cast<int64_t>(c) * taps + k], v, acc);
    }
    stf(y + static_cast<int64_t>(n) * C + c, silu_f(acc));
  }
}

// bf16, 8 channels per thread and a strip of tokens: the window slides through registers. taps <= 4.
constexpr int kStrip = 32;
__global__ void ssm_conv_strip_kernel(const SeqBatch sb, const __nv_bfloat16* __restrict__ x, int64_t ldx,
                                      const float* __restrict__ w, const float* __restrict__ bias,
                                      const float* __restrict__ ring, __nv_bfloat16* __restrict__ y, int C, int taps) {
  const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c0 >= C) return;
  int n = blockIdx.y * kStrip;
  const int n_end = min(n + kStrip, sb.n_tok);
  float wt[8][4], bs[8];   // the last tap (current token) sits in column 3
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    bs[j] = bias[c0 + j];
    if (taps == 4) {
      const float4 v = *reinterpret_cast<const float4*>(w + static_cast<int64_t>(c0 + j) * 4);
      wt[j][0] = v.x; wt[j][1] = v.y; wt[j][2] = v.z; wt[j][3] = v.w;
    } else {
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const int kk = k - (4 - taps);
        wt[j][k] = kk >= 0 ? w[static_cast<int64_t>(c0 + j) * taps + kk] : 0.f;
      }
    }
  }
  float win[3][8];
  int b = -1, seq_end = -1;
#pragma unroll 4
  for (; n < n_end; ++n) {
    if (n >= seq_end) {   // a new sequence starts in this strip, or the strip itself starts: reload the window
      b = sb.tok_seq[n];
      seq_end = sb.cu[b + 1];
      const int first = sb.cu[b], start = sb.start[b], pos = start + n - first;
      const float* rg = ring + static_cast<int64_t>(sb.ids[b]) * taps * C;
#pragma unroll
      for (int k = 0; k < 3; ++k) {
        const int p = pos - 3 + k;
#pragma unroll
        for (int j = 0; j < 8; ++j) win[k][j] = 0.f;
        if (p >= start) {
          Vec16<__nv_bfloat16>::load(x + static_cast<int64_t>(first + p - start) * ldx + c0, win[k]);
        } else if (p >= 0 && p > pos - taps) {
#pragma unroll
          for (int j = 0; j < 8; ++j) win[k][j] = rg[static_cast<int64_t>(p % taps) * C + c0 + j];
        }
      }
    }
    float cur[8];
    Vec16<__nv_bfloat16>::load(x + static_cast<int64_t>(n) * ldx + c0, cur);   // independent of the window: loads run ahead
    uint32_t o[4];
    float r[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      float a = bs[j];
      a = fmaf(wt[j][0], win[0][j], a);
      a = fmaf(wt[j][1], win[1][j], a);
      a = fmaf(wt[j][2], win[2][j], a);
      a = fmaf(wt[j][3], cur[j], a);
      r[j] = __fdividef(a, 1.f + __expf(-a));
      win[0][j] = win[1][j];
      win[1][j] = win[2][j];
      win[2][j] = cur[j];
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) o[j] = pack_bf16x2(r[2 * j], r[2 * j + 1]);
    *reinterpret_cast<uint4*>(y + static_cast<int64_t>(n) * C + c0) = make_uint4(o[0], o[1], o[2], o[3]);
  }
}

template <typename T>
__global__ void ssm_ring_kernel(const SeqBatch sb, const T* __restrict__ x, int64_t ldx, float* __restrict__ ring, int C,
                                int taps) {
  const int b = blockIdx.y;
  const int first = sb.cu[b], len = sb.cu[b + 1] - first, start = sb.start[b];
  float* rg = ring + static_cast<int64_t>(sb.ids[b]) * taps * C;
  const int keep = min(taps - 1, len);
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < keep * C; i += gridDim.x * blockDim.x) {
    const int t = len - keep + i / C, c = i % C;
    rg[static_cast<int64_t>((start + t) % taps) * C + c] = ldf(x + static_cast<int64_t>(first + t) * ldx + c);
  }
}

// ---- recurrence, token by token -----------------------------------------------------------------------------------------
// Block: one head of one sequence, 16 columns of the state; thread (p, g) holds rows g, g + 8, ... of column p.
constexpr int kScanP = 16, kScanG = 8, kScanTok = 16;

template <typename T, int NS>
__global__ void __launch_bounds__(kScanP * kScanG)
ssd_scan_kernel(const SeqBatch sb, const T* __restrict__ xbc, const T* __restrict__ dt_raw, int64_t ld_dt,
                const float* __restrict__ dt_bias, const float* __restrict__ a_log, const float* __restrict__ d_skip,
                float* __restrict__ state, T* __restrict__ y, const SsdShape s) {
  extern __shared__ float sm[];
  const int N = s.N, P = s.P;
  float* sB = sm;                       // [kScanTok][N]
  float* sC = sB + kScanTok * N;        // [kScanTok][N]
  float* sX = sC + kScanTok * N;        // [kScanTok][kScanP]
  float* sDt = sX + kScanTok * kScanP;  // [kScanTok]
  float* sDa = sDt + kScanTok;          // [kScanTok]
  const int h = blockIdx.x, p0 = blockIdx.y * kScanP, b = blockIdx.z;
  const int g = threadIdx.x % kScanG, p = threadIdx.x / kScanG;   // the eight row groups of a column are neighbours
  const int first = sb.cu[b], len = sb.cu[b + 1] - first;
  const int inner = s.H * P, C = inner + 2 * s.G * N;
  const int colB = inner + (h / (s.H / s.G)) * N, colC = colB + s.G * N;
  float* st = state + (static_cast<int64_t>(sb.ids[b]) * s.H + h) * N * P;
  const bool live = p0 + p < P;
  float S[NS];
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = g + i * kScanG;
    S[i] = (sb.start[b] > 0 && live && n < N) ? st[static_cast<int64_t>(n) * P + p0 + p] : 0.f;
  }
  const float bias = dt_bias[h], a = -expf(a_log[h]), dsk = d_skip[h];
  for (int t0 = 0; t0 < len; t0 += kScanTok) {
    const int cnt = min(kScanTok, len - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < cnt * N; i += blockDim.x) {
      const T* row = xbc + static_cast<int64_t>(first + t0 + i / N) * C;
      sB[i] = ldf(row + colB + i % N);
      sC[i] = ldf(row + colC + i % N);
    }
    for (int i = threadIdx.x; i < cnt * kScanP; i += blockDim.x)
      sX[i] = p0 + i % kScanP < P ? ldf(xbc + static_cast<int64_t>(first + t0 + i / kScanP) * C + h * P + p0 + i % kScanP) : 0.f;
    if (threadIdx.x < cnt) {
      const float dt = softplus_f(ldf(dt_raw + static_cast<int64_t>(first + t0 + threadIdx.x) * ld_dt + h) + bias);
      sDt[threadIdx.x] = dt;
      sDa[threadIdx.x] = expf(a * dt);
    }
    __syncthreads();
    for (int t = 0; t < cnt; ++t) {
      const float da = sDa[t], x = sX[t * kScanP + p], dx = sDt[t] * x;
      float acc = 0.f;
#pragma unroll
      for (int i = 0; i < NS; ++i) {
        const int n = g + i * kScanG;
        if (n < N) {
          S[i] = fmaf(S[i], da, dx * sB[t * N + n]);
          acc = fmaf(S[i], sC[t * N + n], acc);
        }
      }
#pragma unroll
      for (int o = 1; o < kScanG; o <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
      if (g == 0 && live) stf(y + static_cast<int64_t>(first + t0 + t) * inner + h * P + p0 + p, fmaf(dsk, x, acc));
    }
  }
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = g + i * kScanG;
    if (live && n < N) st[static_cast<int64_t>(n) * P + p0 + p] = S[i];
  }
}

template <typename T>
cudaError_t ssd_scan_t(const SeqBatch& sb, const T* xbc, const T* dt_raw, int64_t ld_dt, const float* dt_bias,
                       const float* a_log, const float* d_skip, float* state, T* y, const SsdShape& s, cudaStream_t st) {
  const dim3 grid(s.H, (s.P + kScanP - 1) / kScanP, sb.n_seq);
  const int smem = 4 * (2 * kScanTok * s.N + kScanTok * kScanP + 2 * kScanTok);
#define B200_SCAN(NS)                                                                                                  \
  {                                                                                                                    \
    static bool configured = false;                                                                                    \
    if (!configured) {                                                                                                 \
      cudaError_t e = cudaFuncSetAttribute(ssd_scan_kernel<T, NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024); \
      if (e != cudaSuccess) return e;                                                                                  \
      configured = true;                                                                                               \
    }                                                                                                                  \
    ssd_scan_kernel<T, NS><<<grid, kScanP * kScanG, smem, st>>>(sb, xbc, dt_raw, ld_dt, dt_bias, a_log, d_skip, state, y, s); \
  }
  if (s.N <= 64) B200_SCAN(8)
  else if (s.N <= 128) B200_SCAN(16)
  else if (s.N <= 256) B200_SCAN(32)
  else if (s.N <= 512) B200_SCAN(64)
  else return cudaErrorInvalidValue;
#undef B200_SCAN
  return cudaGetLastError();
}

// ---- decode ---------------------------------------------------------------------------------------------------------
// Block: one head of one sequence. Phase 1 convolves the head's x channels and its group's B and C channels (the ring
// row of the new position is nobody's input in this step, so blocks that share a group do not race). Phase 2 streams
// the state: thread (row r, column lane) with `lanes` columns-of-V per row.
constexpr int kDecThreads = 256;

template <typename T, int V>
__global__ void __launch_bounds__(kDecThreads)
ssm_decode_kernel(const SeqBatch sb, const T* __restrict__ zxd, int64_t ldz, const float* __restrict__ w,
                  const float* __restrict__ bias, float* __restrict__ ring, int taps, const float* __restrict__ dt_bias,
                  const float* __restrict__ a_log, const float* __restrict__ d_skip, float* __restrict__ state,
                  float* __restrict__ y, const SsdShape s) {
  extern __shared__ float sm[];
  const int N = s.N, P = s.P;
  float* sx = sm;            // [P]
  float* sB = sx + P;        // [N]
  float* sC = sB + N;        // [N]
  float* red = sC + N;       // [rows][P]
  const int h = blockIdx.x, b = blockIdx.y;
  const int slot = sb.ids[b], pos = sb.start[b];
  const int inner = s.H * P, C = inner + 2 * s.G * N, hpg = s.H / s.G;
  const int grp = h / hpg;
  const T* row = zxd + static_cast<int64_t>(sb.cu[b]) * ldz;
  float* rg = ring + static_cast<int64_t>(slot) * taps * C;
  for (int i = threadIdx.x; i < P + 2 * N; i += blockDim.x) {
    const int c = i < P ? h * P + i : (i < P + N ? inner + grp * N + i - P : inner + s.G * N + grp * N + i - P - N);
    const float cur = ldf(row + inner + c);
    float acc = bias[c];
    for (int k = 0; k < taps - 1; ++k) {
      const int p = pos - (taps - 1) + k;
      if (p >= 0) acc = fmaf(w[static_cast<int64_t>(c) * taps + k], rg[static_cast<int64_t>(p % taps) * C + c], acc);
    }
    acc = fmaf(w[static_cast<int64_t>(c) * taps + taps - 1], cur, acc);
    sm[i] = rnd<T>(silu_f(acc));
    if (i < P || h % hpg == 0) rg[static_cast<int64_t>(pos % taps) * C + c] = cur;
  }
  const float dt = softplus_f(ldf(row + 2 * inner + 2 * s.G * N + h) + dt_bias[h]);
  const float da = expf(-expf(a_log[h]) * dt);
  __syncthreads();
  const int lanes = P / V, rows = kDecThreads / lanes;   // P / V <= kDecThreads (checked by the launcher)
  const int r = threadIdx.x / lanes, c = (threadIdx.x % lanes) * V;
  float* st = state + (static_cast<int64_t>(slot) * s.H + h) * N * P;
  if (r < rows) {
    float acc[V], dx[V];
#pragma unroll
    for (int j = 0; j < V; ++j) { acc[j] = 0.f; dx[j] = dt * sx[c + j]; }
#pragma unroll 4
    for (int n = r; n < N; n += rows) {
      float S[V];
      float* sp = st + static_cast<int64_t>(n) * P + c;
      if (pos > 0) {
        if constexpr (V == 4) {
          const float4 f = *reinterpret_cast<const float4*>(sp);
          S[0] = f.x; S[1] = f.y; S[2] = f.z; S[3] = f.w;
        } else {
          S[0] = sp[0];
        }
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) S[j] = 0.f;
      }
      const float bn = sB[n], cn = sC[n];
#pragma unroll
      for (int j = 0; j < V; ++j) {
        S[j] = fmaf(S[j], da, dx[j] * bn);
        acc[j] = fmaf(S[j], cn, acc[j]);
      }
      if constexpr (V == 4) *reinterpret_cast<float4*>(sp) = make_float4(S[0], S[1], S[2], S[3]);
      else sp[0] = S[0];
    }
#pragma unroll
    for (int j = 0; j < V; ++j) red[r * P + c + j] = acc[j];
  }
  __syncthreads();
  for (int p = threadIdx.x; p < P; p += blockDim.x) {
    float v = 0.f;
    for (int q = 0; q < rows; ++q) v += red[q * P + p];
    v = fmaf(d_skip[h], sx[p], v);
    y[static_cast<int64_t>(b) * inner + h * P + p] = v * silu_f(ldf(row + h * P + p));
  }
}

// ---- gated norm -------------------------------------------------------------------------------------------------------
template <typename TY, typename T>
__global__ void gated_group_norm_kernel(const TY* __restrict__ y, const T* __restrict__ z, int64_t ldz,
                                        const float* __restrict__ gamma, T* __restrict__ out, int D, int part, float eps) {
  extern __shared__ float buf[];   // [part]
  __shared__ float red[33];
  const int n = blockIdx.x, c0 = blockIdx.y * part;
  const TY* yr = y + static_cast<int64_t>(n) * D + c0;
  float ss = 0.f;
  for (int i = threadIdx.x; i < part; i += blockDim.x) {
    float v = ldf(yr + i);
    if (z != nullptr) v *= silu_f(ldf(z + static_cast<int64_t>(n) * ldz + c0 + i));
    buf[i] = v;
    ss += v * v;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / part + eps);
  for (int i = threadIdx.x; i < part; i += blockDim.x)
    stf(out + static_cast<int64_t>(n) * D + c0 + i, buf[i] * inv * gamma[c0 + i]);
}

// bf16 y and z, part <= 8 * kThr * kIt:
// eight features per thread and step; kThr threads (a warp or the block) own one piece of one row
template <int kIt, int kThr>
__global__ void __launch_bounds__(256)
gated_group_norm_vec_kernel(const __nv_bfloat16* __restrict__ y, const __nv_bfloat16* __restrict__ z, int64_t ldz,
                            const float* __restrict__ gamma, __nv_bfloat16* __restrict__ out, int pieces, int parts, int D,
                            int part, float eps) {
  __shared__ float red[33];
  const int piece = blockIdx.x * (256 / kThr) + threadIdx.x / kThr, tid = threadIdx.x % kThr;
  if (kThr == 32 && piece >= pieces) return;
  const int n = piece / parts, c0 = (piece % parts) * part;
  float v[kIt][8];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + tid) * 8;
    if (i < part) {
      float zv[8];
      Vec16<__nv_bfloat16>::load(y + static_cast<int64_t>(n) * D + c0 + i, v[k]);
      Vec16<__nv_bfloat16>::load(z + static_cast<int64_t>(n) * ldz + c0 + i, zv);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        v[k][j] *= __fdividef(zv[j], 1.f + __expf(-zv[j]));
        ss += v[k][j] * v[k][j];
      }
    }
  }
  const float inv = 1.f / sqrtf((kThr == 32 ? warp_sum(ss) : block_sum(ss, red)) / part + eps);
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + tid) * 8;
    if (i < part) {
      const float4 g0 = *reinterpret_cast<const float4*>(gamma + c0 + i), g1 = *reinterpret_cast<const float4*>(gamma + c0 + i + 4);
      *reinterpret_cast<uint4*>(out + static_cast<int64_t>(n) * D + c0 + i) =
          make_uint4(pack_bf16x2(v[k][0] * inv * g0.x, v[k][1] * inv * g0.y), pack_bf16x2(v[k][2] * inv * g0.z, v[k][3] * inv * g0.w),
                     pack_bf16x2(v[k][4] * inv * g1.x, v[k][5] * inv * g1.y), pack_bf16x2(v[k][6] * inv * g1.z, v[k][7] * inv * g1.w));
    }
  }
}

template <typename TY, typename T>
cudaError_t gated_norm_t(const TY* y, const T* z, int64_t ldz, const float* gamma, T* out, int rows, int D, int parts, float eps,
                         cudaStream_t st) {
  const int part = D / parts;
  if (part * 4 > 160 * 1024) return cudaErrorInvalidValue;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(gated_group_norm_kernel<TY, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  const int th = part >= 1024 ? 256 : (part >= 256 ? 128 : 64);
  gated_group_norm_kernel<TY, T><<<dim3(rows, parts), th, part * 4, st>>>(y, z, ldz, gamma, out, D, part, eps);
  return cudaGetLastError();
}

}  // namespace

cudaError_t launch_ssm_conv(bool f32, const SeqBatch& sb, const void* x, int64_t ldx, const float* w, const float* bias,
                            float* ring, void* y, int C, int taps, cudaStream_t st) {
  if (taps < 1) return cudaErrorInvalidValue;
  const int blocks = (C + 255) / 256;
  if (f32) {
    ssm_conv_kernel<float><<<dim3(sb.n_tok, blocks), 256, 0, st>>>(sb, static_cast<const float*>(x), ldx, w, bias, ring,
                                                                  static_cast<float*>(y), C, taps);
    ssm_ring_kernel<float><<<dim3(blocks, sb.n_seq), 256, 0, st>>>(sb, static_cast<const float*>(x), ldx, ring, C, taps);
  } else {
    const __nv_bfloat16* xb = static_cast<const __nv_bfloat16*>(x);
    __nv_bfloat16* yb = static_cast<__nv_bfloat16*>(y);
    if (taps <= 4 && C % 8 == 0 && ldx % 8 == 0 && (reinterpret_cast<uintptr_t>(xb) & 15) == 0)
      ssm_conv_strip_kernel<<<dim3((C / 8 + 127) / 128, (sb.n_tok + kStrip - 1) / kStrip), 128, 0, st>>>(sb, xb, ldx, w, bias,
                                                                                                       ring, yb, C, taps);
    else
      ssm_conv_kernel<__nv_bfloat16><<<dim3(sb.n_tok, blocks), 256, 0, st>>>(sb, xb, ldx, w, bias, ring, yb, C, taps);
    ssm_ring_kernel<__nv_bfloat16><<<dim3(blocks, sb.n_seq), 256, 0, st>>>(sb, xb, ldx, ring, C, taps);
  }
  return cudaGetLastError();
}

cudaError_t launch_ssd_scan(bool f32, const SeqBatch& sb, const void* xbc, const void* dt_raw, int64_t ld_dt,
                            const float* dt_bias, const float* a_log, const float* d_skip, float* state, void* y,
                            const SsdShape& s, cudaStream_t st) {
  if (s.G < 1 || s.H % s.G != 0) return cudaErrorInvalidValue;
  return f32 ? ssd_scan_t<float>(sb, static_cast<const float*>(xbc), static_cast<const float*>(dt_raw), ld_dt, dt_bias, a_log,
                                 d_skip, state, static_cast<float*>(y), s, st)
             : ssd_scan_t<__nv_bfloat16>(sb, static_cast<const __nv_bfloat16*>(xbc), static_cast<const __nv_bfloat16*>(dt_raw), ld_dt,
                                         dt_bias, a_log, d_skip, state, static_cast<__nv_bfloat16*>(y), s, st);
}

cudaError_t launch_ssm_decode(bool f32, const SeqBatch& sb, const void* zxd, int64_t ldz, const float* w, const float* bias,
                              float* ring, int taps, const float* dt_bias, const float* a_log, const float* d_skip,
                              float* state, float* y, const SsdShape& s, cudaStream_t st) {
  if (s.G < 1 || s.H % s.G != 0 || taps < 1) return cudaErrorInvalidValue;
  const int V = s.P % 4 == 0 ? 4 : 1;
  const int lanes = s.P / V;
  if (lanes > kDecThreads) return cudaErrorInvalidValue;
  const int smem = 4 * (s.P + 2 * s.N + (kDecThreads / lanes) * s.P);
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  const dim3 grid(s.H, sb.n_seq);
#define B200_DEC(T, VV)                                                                                                   \
  ssm_decode_kernel<T, VV><<<grid, kDecThreads, smem, st>>>(sb, static_cast<const T*>(zxd), ldz, w, bias, ring, taps, dt_bias, \
                                                            a_log, d_skip, state, y, s)
  if (f32) { if (V == 4) B200_DEC(float, 4); else B200_DEC(float, 1); }
  else { if (V == 4) B200_DEC(__nv_bfloat16, 4); else B200_DEC(__nv_bfloat16, 1); }
#undef B200_DEC
  return cudaGetLastError();
}

cudaError_t launch_gated_group_norm(bool f32, bool y_f32, const void* y, const void* z, int64_t ldz, const float* gamma,
                                    void* out, int rows, int D, int parts, float eps, cudaStream_t st) {
  if (parts < 1 || D % parts != 0) return cudaErrorInvalidValue;
  const int part = D / parts;
  if (f32)
    return gated_norm_t<float, float>(static_cast<const float*>(y), static_cast<const float*>(z), ldz, gamma,
                                      static_cast<float*>(out), rows, D, parts, eps, st);
  __nv_bfloat16* o = static_cast<__nv_bfloat16*>(out);
  const __nv_bfloat16* zb = static_cast<const __nv_bfloat16*>(z);
  if (y_f32) return gated_norm_t<float, __nv_bfloat16>(static_cast<const float*>(y), zb, ldz, gamma, o, rows, D, parts, eps, st);
  const __nv_bfloat16* yb = static_cast<const __nv_bfloat16*>(y);
  if (zb != nullptr && part % 8 == 0 && ldz % 8 == 0 && (reinterpret_cast<uintptr_t>(zb) & 15) == 0 && part <= 16384) {
    const int pieces = rows * parts;
#define B200_GN(IT, THR) \
  gated_group_norm_vec_kernel<IT, THR><<<(pieces + 256 / THR - 1) / (256 / THR), 256, 0, st>>>(yb, zb, ldz, gamma, o, pieces, parts, D, part, eps)
    if (part <= 512) B200_GN(2, 32);
    else if (part <= 1024) B200_GN(4, 32);
    else if (part <= 2048) B200_GN(1, 256);
    else if (part <= 4096) B200_GN(2, 256);
    else B200_GN(8, 256);
#undef B200_GN
    return cudaGetLastError();
  }
  return gated_norm_t<__nv_bfloat16, __nv_bfloat16>(yb, zb, ldz, gamma, o, rows, D, parts, eps, st);
}

}  // namespace b200
