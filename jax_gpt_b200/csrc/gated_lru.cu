// Real-gated linear recurrent unit on packed batches (De et al., "Griffin: Mixing Gated Linear Recurrences with Local Attention
// for Efficient Language Models"):
//   u = causal depthwise convolution of (x + x_bias), per channel
//   r = sigmoid(W_r u + b_r), i = sigmoid(W_i u + b_i) with block-diagonal W_r, W_i
//   log a = -c r, S_t = a S_(t-1) + sqrt(1 - a^2) i u, out = scale S gelu(y + y_bias);   c = 8 softplus(lambda) per channel
//
// Any sizes: gates of eight rows at a time (a warp per channel), then a scan with a thread per channel; one token per sequence:
// all of it in one launch. bf16 prompts: the gates are tensor-core products with channels as rows and tokens as columns, so that a
// warp holds all tokens of a chunk for its 16 channels and scans them in registers; then a scan over the chunks, then the outputs.
//
// Gates, decays and states are fp32. This file is built without fast-math; the tensor-core kernel names its fast intrinsics.
#include "serve_common.cuh"
#include "serve_kernels.cuh"

namespace b200 {

namespace {

__device__ __forceinline__ float gelu_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z)));
}

// raw convolution input of (sequence, position, channel); zero before the start
template <typename T>
__device__ __forceinline__ float conv_input(const LruArgs& a, int first, int start, int slot, int p, int c) {
  if (p < 0) return 0.f;
  if (p >= start) return ldf(static_cast<const T*>(a.x) + static_cast<int64_t>(first + p - start) * a.ldx + c) + a.x_bias[c];
  return a.ring[(static_cast<int64_t>(slot) * a.taps + p % a.taps) * a.W + c];
}
template <typename T>
__device__ __forceinline__ float conv_at(const LruArgs& a, int first, int start, int slot, int pos, int c) {
  float acc = a.conv_bias[c];
  for (int k = 0; k < a.taps; ++k)
    acc = fmaf(a.conv[static_cast<int64_t>(c) * a.taps + k], conv_input<T>(a, first, start, slot, pos - (a.taps - 1) + k, c), acc);
  return acc;
}

// exp(la) S + in as a change of S: decays close to 1 keep their distance from it, whose rounding would add up over a long memory
__device__ __forceinline__ float decayed(float S, float la, float in) { return S + fmaf(expm1f(la), S, in); }

// ---- gates, any sizes; kStep: the whole unit for one token per sequence ----------------------------------------------------
constexpr int kLruTok = 8, kLruWarps = 8;

template <typename T, bool kStep>
__global__ void __launch_bounds__(kLruWarps * 32)
lru_gates_kernel(const SeqBatch sb, const LruArgs a, int per_block, float* __restrict__ log_a, float* __restrict__ inp) {
  extern __shared__ float su[];   // [kLruTok][wb]
  const int wb = a.W / a.blocks, blk = blockIdx.y, n0 = blockIdx.x * kLruTok, cnt = min(kLruTok, sb.n_tok - n0);
  const int c0 = blockIdx.z * per_block, c1 = min(wb, c0 + per_block);
  for (int i = threadIdx.x; i < kLruTok * wb; i += blockDim.x) {
    const int t = i / wb, k = i % wb, n = n0 + t, c = blk * wb + k;
    float u = 0.f;
    if (t < cnt) {
      const int b = sb.tok_seq[n], first = sb.cu[b], start = sb.start[b], pos = start + n - first, slot = sb.ids[b];
      u = conv_at<T>(a, first, start, slot, pos, c);
      // rows of the ring that other blocks may still read belong to the taps - 1 positions before this one
      if (kStep && k >= c0 && k < c1) a.ring[(static_cast<int64_t>(slot) * a.taps + pos % a.taps) * a.W + c] = conv_input<T>(a, first, start, slot, pos, c);
    }
    su[i] = u;
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* w = static_cast<const T*>(a.gates) + static_cast<int64_t>(blk) * 2 * wb * wb;
  for (int k = c0 + warp; k < c1; k += kLruWarps) {
    const T *wr = w + static_cast<int64_t>(k) * wb, *wi = wr + static_cast<int64_t>(wb) * wb;
    float ar[kLruTok], ai[kLruTok];
#pragma unroll
    for (int t = 0; t < kLruTok; ++t) ar[t] = ai[t] = 0.f;
    for (int j = lane; j < wb; j += 32) {
      const float x = ldf(wr + j), z = ldf(wi + j);
#pragma unroll
      for (int t = 0; t < kLruTok; ++t) {
        const float u = su[t * wb + j];
        ar[t] = fmaf(x, u, ar[t]);
        ai[t] = fmaf(z, u, ai[t]);
      }
    }
    float mr = 0.f, mi = 0.f;   // lane t keeps row t
#pragma unroll
    for (int t = 0; t < kLruTok; ++t) {
      const float r = warp_sum(ar[t]), i = warp_sum(ai[t]);
      if (lane == t) { mr = r; mi = i; }
    }
    if (lane >= cnt) continue;
    const int n = n0 + lane, c = blk * wb + k;
    const float r = sigmoid_f(mr + a.gates_bias[(blk * 2) * wb + k]), i = sigmoid_f(mi + a.gates_bias[(blk * 2 + 1) * wb + k]);
    const float la = -a.decay[c] * r, in = sqrtf(-expm1f(2.f * la)) * i * su[lane * wb + k];
    if constexpr (kStep) {
      const int b = sb.tok_seq[n], slot = sb.ids[b];
      float* sp = a.state + static_cast<int64_t>(slot) * a.W + c;
      const float S = decayed(sb.start[b] > 0 ? *sp : 0.f, la, in);
      *sp = S;
      const float y = gelu_f(ldf(static_cast<const T*>(a.y) + static_cast<int64_t>(n) * a.ldy + c) + a.y_bias[c]);
      stf(static_cast<T*>(a.out) + static_cast<int64_t>(n) * a.ldo + c, a.scale * S * y);
    } else {
      log_a[static_cast<int64_t>(n) * a.W + c] = la;
      inp[static_cast<int64_t>(n) * a.W + c] = in;
    }
  }
}

// ---- scan, any sizes: a thread per channel ---------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(64)
lru_scan_kernel(const SeqBatch sb, const LruArgs a, const float* __restrict__ log_a, const float* __restrict__ inp) {
  const int c = blockIdx.x * 64 + threadIdx.x, b = blockIdx.y;
  if (c >= a.W) return;
  const int first = sb.cu[b], end = sb.cu[b + 1];
  float* sp = a.state + static_cast<int64_t>(sb.ids[b]) * a.W + c;
  float S = sb.start[b] > 0 ? *sp : 0.f;
  const float yb = a.y_bias[c];
  constexpr int kAhead = 8;
  for (int n0 = first; n0 < end; n0 += kAhead) {
    float la[kAhead], in[kAhead], y[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      const int64_t n = min(n0 + j, end - 1);
      la[j] = log_a[n * a.W + c];
      in[j] = inp[n * a.W + c];
      y[j] = ldf(static_cast<const T*>(a.y) + n * a.ldy + c);
    }
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      if (n0 + j >= end) break;
      S = decayed(S, la[j], in[j]);
      stf(static_cast<T*>(a.out) + static_cast<int64_t>(n0 + j) * a.ldo + c, a.scale * S * gelu_f(y[j] + yb));
    }
  }
  *sp = S;
}

// the portion's last taps - 1 inputs
template <typename T>
__global__ void lru_ring_kernel(const SeqBatch sb, const LruArgs a) {
  const int b = blockIdx.y, first = sb.cu[b], len = sb.cu[b + 1] - first, start = sb.start[b], keep = min(a.taps - 1, len);
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < keep * a.W; i += gridDim.x * blockDim.x) {
    const int t = len - keep + i / a.W, c = i % a.W;
    a.ring[(static_cast<int64_t>(sb.ids[b]) * a.taps + (start + t) % a.taps) * a.W + c] =
        ldf(static_cast<const T*>(a.x) + static_cast<int64_t>(first + t) * a.ldx + c) + a.x_bias[c];
  }
}

template <typename T>
cudaError_t lru_ring_go(const SeqBatch& sb, const LruArgs& a, cudaStream_t st) {
  const int n = (a.taps - 1) * a.W;
  if (n > 0) lru_ring_kernel<T><<<dim3((n + 255) / 256, sb.n_seq), 256, 0, st>>>(sb, a);
  return cudaGetLastError();
}

template <typename T, bool kStep>
cudaError_t lru_gates_go(const SeqBatch& sb, const LruArgs& a, float* log_a, float* inp, cudaStream_t st) {
  static int have = 0;
  const int wb = a.W / a.blocks, smem = kLruTok * wb * 4, tiles = (sb.n_tok + kLruTok - 1) / kLruTok;
  const cudaError_t e = want_smem(lru_gates_kernel<T, kStep>, smem, have);
  if (e != cudaSuccess) return e;
  int per = wb;   // channels per block: one launch covers the SMs
  while (per > kLruWarps && static_cast<int64_t>(tiles) * a.blocks * ((wb + per - 1) / per) < 148) per = (per + 1) / 2;
  lru_gates_kernel<T, kStep><<<dim3(tiles, a.blocks, (wb + per - 1) / per), kLruWarps * 32, smem, st>>>(sb, a, per, log_a, inp);
  return cudaGetLastError();
}

// ---- bf16 prompts on tensor cores --------------------------------------------------------------------------------------
// lru_chunk: a block per chunk of 64 tokens of one sequence and up to 128 channels of one gate block, a warp per 16 channels. The
// convolved inputs of the whole gate block are staged as rows (token, channel) in a high and a low bf16 part; mma.sync m16n8k16 with
// gate weights as the 16-row operand and tokens as columns (tcgen05 would leave a channel per TMEM lane, and the scan would take it
// back through tcgen05.ld; here the accumulators are where the scan wants them). Column g of tile n is token 16 (g / 2) + 2 n + g % 2,
// so that a lane's 16 columns are 16 consecutive tokens of its two channels: the scan is a loop in the lane and one composition over
// four lanes. Contraction indices are permuted alike on both sides, which leaves the sums unchanged. Every token's composition
// (factor, offset) from the chunk's start goes to memory, the start states follow from a scan over the chunks (lru_prefix), and
// lru_output makes the outputs.
constexpr int kChunk = 64, kSlice = 128, kStripTok = 4;

__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
// a = exp(-x), d = 1 - a and 1 - a^2 for x >= 0, all to fp32 rounding also where a is close to 1
__device__ __forceinline__ void decay_pair(float x, float& d, float& a, float& om) {
  const float p = x * (1.f - x * (0.5f - x * (1.f / 6 - x * (1.f / 24 - x * (1.f / 120)))));
  const float e = ex2_approx(-kLog2e * x);
  d = x < 0.125f ? p : 1.f - e;
  a = x < 0.125f ? 1.f - p : e;
  om = d * (2.f - d);
}
__host__ __device__ __forceinline__ int staged_ld(int wb) {   // row stride of the staged inputs: 64 bytes past a multiple of 128
  const int k = (wb + 31) / 32;
  return (k % 2 == 0 ? k + 1 : k) * 32;
}
// rows turn by 16 bytes every 16 tokens: lanes that read one channel of tokens 16 apart hit different banks
__host__ __device__ __forceinline__ int staged_size(int wb) { return kChunk * staged_ld(wb) + kChunk / 16 * 8; }
__device__ __forceinline__ int staged_row(int tok, int ldu) { return tok * ldu + (tok >> 4) * 8; }

struct ChunkOf {
  int b, t0, cnt;   // sequence, first token in it, tokens
};
__device__ __forceinline__ ChunkOf chunk_of(const SeqBatch& sb, int tile) {
  for (int b = 0; b < sb.n_seq; ++b) {
    const int len = sb.cu[b + 1] - sb.cu[b], n = (len + kChunk - 1) / kChunk;
    if (tile < n) return {b, tile * kChunk, min(kChunk, len - tile * kChunk)};
    tile -= n;
  }
  return {-1, 0, 0};
}

__global__ void __launch_bounds__(kSlice * 2, 2)
lru_chunk_kernel(const SeqBatch sb, const LruArgs a, float2* __restrict__ steps, float2* __restrict__ totals) {
  using B = __nv_bfloat16;
  extern __shared__ __align__(16) unsigned char smem[];
  const ChunkOf ch = chunk_of(sb, blockIdx.x);
  if (ch.b < 0) return;
  const int wb = a.W / a.blocks, ldu = staged_ld(wb), blk = blockIdx.y, c0 = blockIdx.z * kSlice, cc = min(kSlice, wb - c0);
  B* su = reinterpret_cast<B*>(smem);                          // high parts
  B* sl = su + staged_size(wb);                                // low parts
  float* sw = reinterpret_cast<float*>(sl + staged_size(wb));  // [3 + taps][wb]: x_bias, conv_bias, conv_bias + sum(conv) x_bias, taps
  const int first = sb.cu[ch.b], start = sb.start[ch.b], slot = sb.ids[ch.b];
  const B* x = static_cast<const B*>(a.x);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3, cw = c0 + warp * 16;
  const B* wr = static_cast<const B*>(a.gates) + (static_cast<int64_t>(blk) * 2 * wb + min(cw, wb - 16) + g) * wb;
  const B* wi = wr + static_cast<int64_t>(wb) * wb;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  struct Weights {
    uint4 r0, r1, i0, i1;
  };
  auto weights = [&](int kb) {
    const int k = kb + t * 8;
    if (k >= wb) return Weights{zero, zero, zero, zero};
    return Weights{__ldg(reinterpret_cast<const uint4*>(wr + k)), __ldg(reinterpret_cast<const uint4*>(wr + 8 * wb + k)),
                   __ldg(reinterpret_cast<const uint4*>(wi + k)), __ldg(reinterpret_cast<const uint4*>(wi + 8 * wb + k))};
  };
  for (int i = threadIdx.x; i < wb; i += blockDim.x) {
    const int c = blk * wb + i;
    const float xb = a.x_bias[c], cb = a.conv_bias[c];
    float sum = 0.f;
    for (int k = 0; k < a.taps; ++k) {
      const float w = a.conv[static_cast<int64_t>(c) * a.taps + k];
      sw[(3 + k) * wb + i] = w;
      sum += w;
    }
    sw[i] = xb;
    sw[wb + i] = cb;
    sw[2 * wb + i] = fmaf(sum, xb, cb);
  }
  // ---- convolution: four tokens of eight channels at a time ----
  const int groups = wb / 8;
  auto put = [&](int tok, int k8, const float (&v)[8]) {
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      hi[j] = pack_bf16x2(v[2 * j], v[2 * j + 1]);
      const float2 h = unpack_bf16x2(hi[j]);
      lo[j] = pack_bf16x2(v[2 * j] - h.x, v[2 * j + 1] - h.y);
    }
    const int at = staged_row(tok, ldu) + k8;
    *reinterpret_cast<uint4*>(su + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(sl + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  };
  const int items = groups * (kChunk / kStripTok);
  uint4 raw[7];   // inputs of tokens -3 .. 3 of this thread's first strip, loaded ahead of the barrier
  auto fetch = [&](int i) {
    const int k8 = i % groups * 8, t0 = i / groups * kStripTok;
    const B* xr = x + static_cast<int64_t>(first + ch.t0) * a.ldx + blk * wb + k8;
#pragma unroll
    for (int k = 0; k < 7; ++k) {
      const int r = t0 - 3 + k;
      raw[k] = r > t0 - a.taps && r < ch.cnt && ch.t0 + r >= 0 ? *reinterpret_cast<const uint4*>(xr + static_cast<int64_t>(r) * a.ldx) : zero;
    }
  };
  if (threadIdx.x < items) fetch(threadIdx.x);
  __syncthreads();
  for (int i = threadIdx.x; i < items; i += blockDim.x) {
    if (i != threadIdx.x) fetch(i);
    const int k8 = i % groups * 8, t0 = i / groups * kStripTok, c = blk * wb + k8;
    if (a.taps <= 4 && ch.t0 + t0 >= a.taps - 1) {     // every input lies in this portion
      float w[4][8], cb[8];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const int kk = k - (4 - a.taps);
        if (kk >= 0) {
          load8(sw + (3 + kk) * wb + k8, w[k]);
        } else {
#pragma unroll
          for (int j = 0; j < 8; ++j) w[k][j] = 0.f;
        }
      }
      load8(sw + 2 * wb + k8, cb);
      float v[kStripTok][8];
#pragma unroll
      for (int q = 0; q < kStripTok; ++q)
#pragma unroll
        for (int j = 0; j < 8; ++j) v[q][j] = cb[j];
#pragma unroll
      for (int k = 0; k < 7; ++k) {
        const uint32_t u[4] = {raw[k].x, raw[k].y, raw[k].z, raw[k].w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 f = unpack_bf16x2(u[j]);
#pragma unroll
          for (int q = 0; q < kStripTok; ++q)
            if (k - q >= 0 && k - q < 4) {
              v[q][2 * j] = fmaf(w[k - q][2 * j], f.x, v[q][2 * j]);
              v[q][2 * j + 1] = fmaf(w[k - q][2 * j + 1], f.y, v[q][2 * j + 1]);
            }
        }
      }
#pragma unroll
      for (int q = 0; q < kStripTok; ++q) put(t0 + q, k8, v[q]);
    } else {
      for (int q = 0; q < kStripTok; ++q) {
        float acc[8], xb[8];
        load8(sw + wb + k8, acc);
        load8(sw + k8, xb);
        for (int k = 0; k < a.taps; ++k) {
          const int p = start + ch.t0 + min(t0 + q, ch.cnt - 1) - (a.taps - 1) + k;
          if (p < 0) continue;
          float v[8], w[8];
          load8(sw + (3 + k) * wb + k8, w);
          if (p >= start) {
            Vec16<B>::load(x + static_cast<int64_t>(first + p - start) * a.ldx + c, v);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] += xb[j];
          } else {
            load8(a.ring + (static_cast<int64_t>(slot) * a.taps + p % a.taps) * a.W + c, v);
          }
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[j] = fmaf(w[j], v[j], acc[j]);
        }
        put(t0 + q, k8, acc);
      }
    }
  }
  const int tail = (ldu - wb) / 8;   // the contraction's tail
  for (int i = threadIdx.x; i < kChunk * tail; i += blockDim.x) {
    const int at = staged_row(i / tail, ldu) + wb + (i % tail) * 8;
    *reinterpret_cast<uint4*>(su + at) = zero;
    *reinterpret_cast<uint4*>(sl + at) = zero;
  }
  Weights next = weights(0);
  __syncthreads();
  if (warp * 16 >= cc) return;
  // ---- gates ----
  float r[8][4], v[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) r[n][j] = v[n][j] = 0.f;
  const int ub = staged_row((g >> 1) * 16 + (g & 1), ldu);
  for (int kb = 0; kb < wb; kb += 32) {
    const Weights w = next;
    if (kb + 32 < wb) next = weights(kb + 32);
#pragma unroll
    for (int part = 0; part < 2; ++part) {
      const B* u0 = (part == 0 ? su : sl) + ub + kb + t * 8;
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        const uint4 u = *reinterpret_cast<const uint4*>(u0 + 2 * n * ldu);
        mma_bf16_16816(r[n], w.r0.x, w.r1.x, w.r0.y, w.r1.y, u.x, u.y);
        mma_bf16_16816(v[n], w.i0.x, w.i1.x, w.i0.y, w.i1.y, u.x, u.y);
        mma_bf16_16816(r[n], w.r0.z, w.r1.z, w.r0.w, w.r1.w, u.z, u.w);
        mma_bf16_16816(v[n], w.i0.z, w.i1.z, w.i0.w, w.i1.w, u.z, u.w);
      }
    }
  }
  // ---- decays and inputs, scan: element j of tile n is channel g + 8 (j / 2), token 16 t + 2 n + j % 2 ----
  const int live = ch.cnt - 16 * t;   // tokens of this lane
  float2* sp = steps + static_cast<int64_t>(first + ch.t0 + 16 * t) * a.W;
  const int ut = staged_row(16 * t, ldu);
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int cb = cw + g + 8 * h, c = blk * wb + cb;
    const float br = a.gates_bias[(blk * 2) * wb + cb], bi = a.gates_bias[(blk * 2 + 1) * wb + cb], dec = a.decay[c];
    float P = 1.f, Q = 0.f;
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int j = 2 * n + e;
        float d, al, om;
        decay_pair(dec * sigmoid_approx(r[n][2 * h + e] + br), d, al, om);
        const float u = __bfloat162float(su[ut + j * ldu + cb]) + __bfloat162float(sl[ut + j * ldu + cb]);
        float in = sqrt_approx(om) * sigmoid_approx(v[n][2 * h + e] + bi) * u;
        if (j >= live) { al = 1.f; in = 0.f; }
        P *= al;
        Q = fmaf(al, Q, in);
        r[n][2 * h + e] = P;       // compositions from the lane's first token on
        v[n][2 * h + e] = Q;
      }
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {
      const float Po = __shfl_up_sync(0xffffffffu, P, o, 4), Qo = __shfl_up_sync(0xffffffffu, Q, o, 4);
      if (t >= o) {
        Q = fmaf(P, Qo, Q);
        P *= Po;
      }
    }
    float Pe = __shfl_up_sync(0xffffffffu, P, 1, 4), Qe = __shfl_up_sync(0xffffffffu, Q, 1, 4);
    if (t == 0) { Pe = 1.f; Qe = 0.f; }
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (2 * n + e < live)
          sp[static_cast<int64_t>(2 * n + e) * a.W + c] = make_float2(r[n][2 * h + e] * Pe, fmaf(r[n][2 * h + e], Qe, v[n][2 * h + e]));
    if (t == 3) totals[static_cast<int64_t>(blockIdx.x) * a.W + c] = make_float2(P, Q);
  }
}

// Start state of every chunk from the chunks' compositions; the slot gets the state after the last one.
__global__ void __launch_bounds__(64)
lru_prefix_kernel(const SeqBatch sb, const LruArgs a, const float2* __restrict__ totals, float* __restrict__ starts) {
  const int c = blockIdx.x * 64 + threadIdx.x, b = blockIdx.y;
  if (c >= a.W) return;
  int64_t tile = 0;
  for (int i = 0; i < b; ++i) tile += (sb.cu[i + 1] - sb.cu[i] + kChunk - 1) / kChunk;
  const int n = (sb.cu[b + 1] - sb.cu[b] + kChunk - 1) / kChunk;
  float* sp = a.state + static_cast<int64_t>(sb.ids[b]) * a.W + c;
  float S = sb.start[b] > 0 ? *sp : 0.f;
  const float2* src = totals + tile * a.W + c;
  float* dst = starts + tile * a.W + c;
  constexpr int kAhead = 32;
  int i = 0;
  for (; i + kAhead <= n; i += kAhead) {
    float2 v[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j) v[j] = __ldcg(src + static_cast<int64_t>(i + j) * a.W);
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      dst[static_cast<int64_t>(i + j) * a.W] = S;
      S = fmaf(v[j].x, S, v[j].y);
    }
  }
  for (; i < n; ++i) {
    const float2 v = __ldcg(src + static_cast<int64_t>(i) * a.W);
    dst[static_cast<int64_t>(i) * a.W] = S;
    S = fmaf(v.x, S, v.y);
  }
  *sp = S;
}

// Outputs: S = factor * start + offset per token and channel, eight channels per thread; a block per 16 tokens of a chunk.
__global__ void __launch_bounds__(256)
lru_output_kernel(const SeqBatch sb, const LruArgs a, const float2* __restrict__ steps, const float* __restrict__ starts) {
  using B = __nv_bfloat16;
  const ChunkOf ch = chunk_of(sb, blockIdx.x);
  if (ch.b < 0) return;
  const int c = (blockIdx.z * 32 + (threadIdx.x & 31)) * 8;
  if (c >= a.W) return;
  float S0[8], yb[8];
  load8(starts + static_cast<int64_t>(blockIdx.x) * a.W + c, S0);
  load8(a.y_bias + c, yb);
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    const int tok = blockIdx.y * 16 + q * 8 + (threadIdx.x >> 5);
    if (tok >= ch.cnt) return;
    const int64_t n = sb.cu[ch.b] + ch.t0 + tok;
    const float4* p = reinterpret_cast<const float4*>(steps + n * a.W + c);
    float y[8];
    Vec16<B>::load(static_cast<const B*>(a.y) + n * a.ldy + c, y);
#pragma unroll
    for (int j = 0; j < 8; j += 2) {
      const float4 f = __ldcs(p + j / 2);
      const float s[2] = {fmaf(f.x, S0[j], f.y), fmaf(f.z, S0[j + 1], f.w)};
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float z = y[j + e] + yb[j + e];
        // z (1 + tanh(w)) / 2 = z / (1 + exp(-2 w))
        y[j + e] = a.scale * s[e] * z * sigmoid_approx(1.5957691216057308f * fmaf(0.044715f * z * z, z, z));
      }
    }
    *reinterpret_cast<uint4*>(static_cast<B*>(a.out) + n * a.ldo + c) =
        make_uint4(pack_bf16x2(y[0], y[1]), pack_bf16x2(y[2], y[3]), pack_bf16x2(y[4], y[5]), pack_bf16x2(y[6], y[7]));
  }
}

// ---- bf16, one token per sequence ----------------------------------------------------------------------------------------
// Block: 16 channels and up to eight sequences (the columns of the gates' products); its four warps split the contraction. Everything
// that does not depend on the gates is loaded first.
__global__ void __launch_bounds__(128)
lru_step_kernel(const SeqBatch sb, const LruArgs a) {
  using B = __nv_bfloat16;
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ float red[4][2][32][4];
  const int wb = a.W / a.blocks, ldu = staged_ld(wb), ch0 = blockIdx.x * 16, blk = ch0 / wb, k0 = ch0 % wb, n0 = blockIdx.y * 8;
  B* su = reinterpret_cast<B*>(smem);   // [8][ldu] high parts
  B* sl = su + 8 * ldu;                 // [8][ldu] low parts
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const B* wr = static_cast<const B*>(a.gates) + (static_cast<int64_t>(blk) * 2 * wb + k0 + g) * wb;
  const B* wi = wr + static_cast<int64_t>(wb) * wb;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  uint4 w[4];
  auto weights = [&](int kb) {
    const int k = kb + t * 8;
    const bool in = k < wb;
    w[0] = in ? __ldg(reinterpret_cast<const uint4*>(wr + k)) : zero;
    w[1] = in ? __ldg(reinterpret_cast<const uint4*>(wr + 8 * wb + k)) : zero;
    w[2] = in ? __ldg(reinterpret_cast<const uint4*>(wi + k)) : zero;
    w[3] = in ? __ldg(reinterpret_cast<const uint4*>(wi + 8 * wb + k)) : zero;
  };
  weights(warp * 32);
  // this thread's output: channel c of sequence n
  const int n = n0 + threadIdx.x / 16, kc = k0 + threadIdx.x % 16, c = blk * wb + kc;
  const bool live = n < sb.n_seq;
  const int slot = live ? sb.ids[n] : 0, pos = live ? sb.start[n] : 0;
  float* sp = a.state + static_cast<int64_t>(slot) * a.W + c;
  const float S0 = live && pos > 0 ? *sp : 0.f;
  const float yv = live ? ldf(static_cast<const B*>(a.y) + static_cast<int64_t>(n) * a.ldy + c) + a.y_bias[c] : 0.f;
  const float xv = live ? ldf(static_cast<const B*>(a.x) + static_cast<int64_t>(n) * a.ldx + c) + a.x_bias[c] : 0.f;
  const float br = a.gates_bias[blk * 2 * wb + kc], bi = a.gates_bias[(blk * 2 + 1) * wb + kc], dec = a.decay[c];
  for (int i = threadIdx.x; i < 8 * (ldu / 8); i += 128) {
    const int q = i / (ldu / 8), k8 = i % (ldu / 8) * 8, m = n0 + q, cc = blk * wb + k8;
    uint32_t hi[4] = {0u, 0u, 0u, 0u}, lo[4] = {0u, 0u, 0u, 0u};
    if (k8 < wb && m < sb.n_seq) {
      const int sm = sb.ids[m], pm = sb.start[m];
      float acc[8], xb[8], v[8];
      load8(a.conv_bias + cc, acc);
      load8(a.x_bias + cc, xb);
      Vec16<B>::load(static_cast<const B*>(a.x) + static_cast<int64_t>(m) * a.ldx + cc, v);
      const float* cw = a.conv + static_cast<int64_t>(cc) * a.taps;
      if (a.taps == 4) {
        float r[3][8];
#pragma unroll
        for (int k = 0; k < 3; ++k) {
#pragma unroll
          for (int j = 0; j < 8; ++j) r[k][j] = 0.f;
          if (pm - 3 + k >= 0) load8(a.ring + (static_cast<int64_t>(sm) * 4 + (pm - 3 + k) % 4) * a.W + cc, r[k]);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const float4 f = *reinterpret_cast<const float4*>(cw + 4 * j);
          acc[j] = fmaf(f.x, r[0][j], fmaf(f.y, r[1][j], fmaf(f.z, r[2][j], fmaf(f.w, v[j] + xb[j], acc[j]))));
        }
      } else {
        for (int k = 0; k + 1 < a.taps; ++k) {
          const int p = pm - (a.taps - 1) + k;
          if (p < 0) continue;
          float r[8];
          load8(a.ring + (static_cast<int64_t>(sm) * a.taps + p % a.taps) * a.W + cc, r);
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[j] = fmaf(cw[j * a.taps + k], r[j], acc[j]);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j] = fmaf(cw[j * a.taps + a.taps - 1], v[j] + xb[j], acc[j]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        hi[j] = pack_bf16x2(acc[2 * j], acc[2 * j + 1]);
        const float2 h = unpack_bf16x2(hi[j]);
        lo[j] = pack_bf16x2(acc[2 * j] - h.x, acc[2 * j + 1] - h.y);
      }
    }
    *reinterpret_cast<uint4*>(su + q * ldu + k8) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(sl + q * ldu + k8) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  __syncthreads();
  float r[4] = {0.f, 0.f, 0.f, 0.f}, v[4] = {0.f, 0.f, 0.f, 0.f};
  for (int kb = warp * 32; kb < wb; kb += 128) {
    if (kb != warp * 32) weights(kb);
#pragma unroll
    for (int part = 0; part < 2; ++part) {
      const uint4 u = *reinterpret_cast<const uint4*>((part == 0 ? su : sl) + g * ldu + kb + t * 8);
      mma_bf16_16816(r, w[0].x, w[1].x, w[0].y, w[1].y, u.x, u.y);
      mma_bf16_16816(v, w[2].x, w[3].x, w[2].y, w[3].y, u.x, u.y);
      mma_bf16_16816(r, w[0].z, w[1].z, w[0].w, w[1].w, u.z, u.w);
      mma_bf16_16816(v, w[2].z, w[3].z, w[2].w, w[3].w, u.z, u.w);
    }
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    red[warp][0][lane][j] = r[j];
    red[warp][1][lane][j] = v[j];
  }
  __syncthreads();
  if (!live) return;
  // accumulator j of lane (g, t): channel g + 8 (j / 2), sequence 2 t + j % 2
  const int q = threadIdx.x / 16, ci = threadIdx.x % 16, src = (ci % 8) * 4 + q / 2, j = (ci / 8) * 2 + q % 2;
  float zr = br, zi = bi;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    zr += red[k][0][src][j];
    zi += red[k][1][src][j];
  }
  const float u = __bfloat162float(su[q * ldu + kc]) + __bfloat162float(sl[q * ldu + kc]);
  float d, al, om;
  decay_pair(dec * sigmoid_approx(zr), d, al, om);
  const float S = S0 + fmaf(-d, S0, sqrt_approx(om) * sigmoid_approx(zi) * u);
  *sp = S;
  a.ring[(static_cast<int64_t>(slot) * a.taps + pos % a.taps) * a.W + c] = xv;   // not a row that the other blocks read
  const float gelu = yv * sigmoid_approx(1.5957691216057308f * fmaf(0.044715f * yv * yv, yv, yv));
  stf(static_cast<B*>(a.out) + static_cast<int64_t>(n) * a.ldo + c, a.scale * S * gelu);
}

bool lru_chunks_ok(const LruArgs& a) {
  const int wb = a.W / a.blocks;
  return wb % 16 == 0 && wb <= 512 && a.taps <= 8 && ((a.ldx | a.ldy | a.ldo) & 7) == 0 &&
         ((reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.out) | reinterpret_cast<uintptr_t>(a.y_bias) |
           reinterpret_cast<uintptr_t>(a.x_bias) | reinterpret_cast<uintptr_t>(a.conv) | reinterpret_cast<uintptr_t>(a.conv_bias) |
           reinterpret_cast<uintptr_t>(a.gates) | reinterpret_cast<uintptr_t>(a.ring)) & 15) == 0;
}

// scratch: steps [n_tok, W] float2, totals [tiles, W] float2, starts [tiles, W], with tiles = n_tok / 64 + n_seq
cudaError_t lru_chunks_go(const SeqBatch& sb, const LruArgs& a, float* scratch, cudaStream_t st) {
  const int wb = a.W / a.blocks, tiles = sb.n_tok / kChunk + sb.n_seq, threads = min(wb, kSlice) * 2;
  const int smem = 2 * staged_size(wb) * 2 + (3 + a.taps) * wb * 4;
  static int have = 0;
  const cudaError_t e = want_smem(lru_chunk_kernel, smem, have);
  if (e != cudaSuccess) return e;
  float2* steps = reinterpret_cast<float2*>(scratch);
  float2* totals = steps + static_cast<int64_t>(sb.n_tok) * a.W;
  float* starts = reinterpret_cast<float*>(totals + static_cast<int64_t>(tiles) * a.W);
  lru_chunk_kernel<<<dim3(tiles, a.blocks, (wb + kSlice - 1) / kSlice), threads, smem, st>>>(sb, a, steps, totals);
  lru_prefix_kernel<<<dim3((a.W + 63) / 64, sb.n_seq), 64, 0, st>>>(sb, a, totals, starts);
  lru_output_kernel<<<dim3(tiles, kChunk / 16, (a.W + 255) / 256), 256, 0, st>>>(sb, a, steps, starts);
  return lru_ring_go<__nv_bfloat16>(sb, a, st);
}

template <typename T>
cudaError_t lru_t(const SeqBatch& sb, const LruArgs& a, float* scratch, cudaStream_t st) {
  if constexpr (sizeof(T) == 2) {
    if (lru_chunks_ok(a)) {
      if (scratch != nullptr) return lru_chunks_go(sb, a, scratch, st);
      lru_step_kernel<<<dim3(a.W / 16, (sb.n_seq + 7) / 8), 128, 2 * 8 * staged_ld(a.W / a.blocks) * 2, st>>>(sb, a);
      return cudaGetLastError();
    }
  }
  if (scratch == nullptr) return lru_gates_go<T, true>(sb, a, nullptr, nullptr, st);
  float *log_a = scratch, *inp = scratch + static_cast<int64_t>(sb.n_tok) * a.W;
  const cudaError_t e = lru_gates_go<T, false>(sb, a, log_a, inp, st);
  if (e != cudaSuccess) return e;
  lru_scan_kernel<T><<<dim3((a.W + 63) / 64, sb.n_seq), 64, 0, st>>>(sb, a, log_a, inp);
  return lru_ring_go<T>(sb, a, st);
}

}  // namespace

int64_t gated_lru_scratch(bool f32, const SeqBatch& sb, const LruArgs& a) {
  const int64_t tiles = sb.n_tok / kChunk + sb.n_seq;
  return (2 * static_cast<int64_t>(sb.n_tok) + (!f32 && lru_chunks_ok(a) ? 3 * tiles : 0)) * a.W;
}

cudaError_t launch_gated_lru(bool f32, const SeqBatch& sb, const LruArgs& a, float* scratch, cudaStream_t st) {
  if (a.blocks < 1 || a.W % a.blocks != 0 || a.taps < 1 || (scratch == nullptr && sb.n_tok != sb.n_seq)) return cudaErrorInvalidValue;
  return f32 ? lru_t<float>(sb, a, scratch, st) : lru_t<__nv_bfloat16>(sb, a, scratch, st);
}

}  // namespace b200
