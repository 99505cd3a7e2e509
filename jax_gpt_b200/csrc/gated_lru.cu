// Real-gated linear recurrent unit on packed batches (De et al., "Griffin: Mixing Gated Linear Recurrences with Local Attention
// for Efficient Language Models"):
//   u = causal depthwise convolution of (x + x_bias), per channel
//   r = sigmoid(W_r u + b_r), i = sigmoid(W_i u + b_i) with block-diagonal W_r, W_i
//   log a = -c r, S_t = a S_(t-1) + sqrt(1 - a^2) i u, out = scale S gelu(y + y_bias);   c = 8 softplus(lambda) per channel
//
// Any sizes: gates of eight rows at a time (a warp per channel), then a scan with a thread per channel; one token per sequence:
// all of it in one launch. bf16 prompts: the gates are tensor-core products with channels as rows and tokens as columns, so that a
// warp holds all tokens of a chunk for its 16 channels and scans them in registers; chunk totals first, then a scan over the
// chunks, then the outputs.
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
      const float S = fmaf(expf(la), sb.start[b] > 0 ? *sp : 0.f, in);
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
      S = fmaf(expf(la[j]), S, in[j]);
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
// Block: a chunk of 64 tokens of one sequence and up to 128 channels of one gate block, a warp per 16 channels. The convolved
// inputs of the whole gate block are staged as rows (token, channel) in a high and a low bf16 part; mma.sync m16n8k16 with gate weights as the 16-row
// operand and tokens as columns (tcgen05 would need both products of 16 channels spread over TMEM lanes, one channel a lane, and
// the scan back through tcgen05.ld; here the accumulators are where the scan wants them). Column g of tile n is token
// 16 (g / 2) + 2 n + g % 2, so that a lane's 16 columns are 16 consecutive tokens of its two channels: the scan is a loop in the
// lane and one composition over four lanes. Contraction indices are permuted alike on both sides, which leaves the sums unchanged.
constexpr int kChunk = 64, kSlice = 128;

__device__ __forceinline__ void mma_16816(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ float fast_sigmoid(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
// 1 - exp(-x) for x >= 0, with e = exp(-x / 2)
__device__ __forceinline__ float one_minus_exp(float x, float e) {
  const float p = x * (1.f - x * (0.5f - x * (1.f / 6 - x * (1.f / 24 - x * (1.f / 120 - x * (1.f / 720))))));
  return x < 0.25f ? p : 1.f - e * e;
}
__host__ __device__ __forceinline__ int staged_ld(int wb) {   // row stride of the staged inputs: 64 bytes past a multiple of 128
  const int k = (wb + 31) / 32;
  return (k % 2 == 0 ? k + 1 : k) * 32;
}

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

// kFinal: outputs from the chunk's start state `starts`; otherwise the chunk's composition (factor, offset) to `totals`.
template <bool kFinal>
__global__ void __launch_bounds__(kSlice * 2, 2)
lru_chunk_kernel(const SeqBatch sb, const LruArgs a, float2* __restrict__ totals, const float* __restrict__ starts) {
  using B = __nv_bfloat16;
  extern __shared__ __align__(16) unsigned char smem[];
  const ChunkOf ch = chunk_of(sb, blockIdx.x);
  if (ch.b < 0) return;
  const int wb = a.W / a.blocks, ldu = staged_ld(wb), blk = blockIdx.y, c0 = blockIdx.z * kSlice, cc = min(kSlice, wb - c0);
  B* su = reinterpret_cast<B*>(smem);                                    // [kChunk][ldu] high parts
  B* sl = su + kChunk * ldu;                                             // [kChunk][ldu] low parts
  float* sw = reinterpret_cast<float*>(sl + kChunk * ldu);               // [2 + taps][wb], later
  float* sS = sw;                                                        // [kChunk][cc] (kFinal)
  const int first = sb.cu[ch.b], start = sb.start[ch.b], slot = sb.ids[ch.b];
  const B* x = static_cast<const B*>(a.x);
  // ---- convolution: eight channels of a token at a time; biases and taps are staged as rows ----
  for (int i = threadIdx.x; i < wb; i += blockDim.x) {
    const int c = blk * wb + i;
    sw[i] = a.x_bias[c];
    sw[wb + i] = a.conv_bias[c];
    for (int k = 0; k < a.taps; ++k) sw[(2 + k) * wb + i] = a.conv[static_cast<int64_t>(c) * a.taps + k];
  }
  __syncthreads();
  const int groups = wb / 8;
  for (int i = threadIdx.x; i < groups * kChunk; i += blockDim.x) {
    const int k8 = i % groups * 8, tok = i / groups, c = blk * wb + k8;
    uint32_t hi[4] = {0u, 0u, 0u, 0u}, lo[4] = {0u, 0u, 0u, 0u};
    if (tok < ch.cnt) {
      float xb[8], acc[8];
      load8(sw + k8, xb);
      load8(sw + wb + k8, acc);
      for (int k = 0; k < a.taps; ++k) {
        const int p = start + ch.t0 + tok - (a.taps - 1) + k;
        if (p < 0) continue;
        float v[8], w[8];
        load8(sw + (2 + k) * wb + k8, w);
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
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        hi[j] = pack_bf16x2(acc[2 * j], acc[2 * j + 1]);
        const float2 h = unpack_bf16x2(hi[j]);
        lo[j] = pack_bf16x2(acc[2 * j] - h.x, acc[2 * j + 1] - h.y);
      }
    }
    *reinterpret_cast<uint4*>(su + tok * ldu + k8) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(sl + tok * ldu + k8) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  for (int i = threadIdx.x; i < kChunk * ((ldu - wb) / 8); i += blockDim.x) {   // the contraction's tail
    const int per = (ldu - wb) / 8;
    *reinterpret_cast<uint4*>(su + (i / per) * ldu + wb + (i % per) * 8) = make_uint4(0u, 0u, 0u, 0u);
    *reinterpret_cast<uint4*>(sl + (i / per) * ldu + wb + (i % per) * 8) = make_uint4(0u, 0u, 0u, 0u);
  }
  __syncthreads();
  // ---- gates ----
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3, cw = c0 + warp * 16;
  if (warp * 16 < cc) {
    float r[8][4], v[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j) r[n][j] = v[n][j] = 0.f;
    const B* wr = static_cast<const B*>(a.gates) + (static_cast<int64_t>(blk) * 2 * wb + cw + g) * wb;
    const B* wi = wr + static_cast<int64_t>(wb) * wb;
    const B* ub = su + ((g >> 1) * 16 + (g & 1)) * ldu;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    for (int kb = 0; kb < wb; kb += 32) {
      const int k = kb + t * 8;
      const bool in = k < wb;
      const uint4 r0 = in ? __ldg(reinterpret_cast<const uint4*>(wr + k)) : zero, r1 = in ? __ldg(reinterpret_cast<const uint4*>(wr + 8 * wb + k)) : zero;
      const uint4 i0 = in ? __ldg(reinterpret_cast<const uint4*>(wi + k)) : zero, i1 = in ? __ldg(reinterpret_cast<const uint4*>(wi + 8 * wb + k)) : zero;
#pragma unroll
      for (int n = 0; n < 8; ++n) {
#pragma unroll
        for (int part = 0; part < 2; ++part) {
          const uint4 u = *reinterpret_cast<const uint4*>(ub + (part * kChunk + 2 * n) * ldu + k);
          mma_16816(r[n], r0.x, r1.x, r0.y, r1.y, u.x, u.y);
          mma_16816(v[n], i0.x, i1.x, i0.y, i1.y, u.x, u.y);
          mma_16816(r[n], r0.z, r1.z, r0.w, r1.w, u.z, u.w);
          mma_16816(v[n], i0.z, i1.z, i0.w, i1.w, u.z, u.w);
        }
      }
    }
    // ---- decays and inputs, scan: element j of tile n is channel g + 8 (j / 2), token 16 t + 2 n + j % 2 ----
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int cb = cw + g + 8 * h, c = blk * wb + cb;
      const float br = a.gates_bias[(blk * 2) * wb + cb], bi = a.gates_bias[(blk * 2 + 1) * wb + cb], dec = a.decay[c];
      float P = 1.f, Q = 0.f;
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int tok = 16 * t + 2 * n + e;
          const float la = -dec * fast_sigmoid(r[n][2 * h + e] + br);
          float al = expf(la);
          const float om = one_minus_exp(-2.f * la, al);
          float in = sqrtf(om) * fast_sigmoid(v[n][2 * h + e] + bi) * (__bfloat162float(su[tok * ldu + cb]) + __bfloat162float(sl[tok * ldu + cb]));
          if (tok >= ch.cnt) { al = 1.f; in = 0.f; }
          r[n][2 * h + e] = al;
          v[n][2 * h + e] = in;
          P *= al;
          Q = fmaf(al, Q, in);
        }
#pragma unroll
      for (int o = 1; o < 4; o <<= 1) {
        const float Po = __shfl_up_sync(0xffffffffu, P, o, 4), Qo = __shfl_up_sync(0xffffffffu, Q, o, 4);
        if (t >= o) {
          Q = fmaf(P, Qo, Q);
          P *= Po;
        }
      }
      const int64_t at = static_cast<int64_t>(blockIdx.x) * a.W + c;
      if constexpr (!kFinal) {
        if (t == 3) totals[at] = make_float2(P, Q);
      } else {
        const float Pe = __shfl_up_sync(0xffffffffu, P, 1, 4), Qe = __shfl_up_sync(0xffffffffu, Q, 1, 4), S0 = starts[at];
        float S = t > 0 ? fmaf(Pe, S0, Qe) : S0;
        int col = warp * 16 + g + 8 * h + 8 * t;   // columns of a row turn by 8 every 16 tokens: the lanes hit different banks
        if (col >= cc) col -= cc;
        if (col >= cc) col -= cc;
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            S = fmaf(r[n][2 * h + e], S, v[n][2 * h + e]);
            sS[(16 * t + 2 * n + e) * cc + col] = S;
          }
      }
    }
  }
  if constexpr (kFinal) {
    __syncthreads();
    // ---- output gate ----
    const int per = cc / 8;
    for (int i = threadIdx.x; i < ch.cnt * per; i += blockDim.x) {
      const int tok = i / per, c8 = i % per * 8, c = blk * wb + c0 + c8;
      const int64_t n = first + ch.t0 + tok;
      int col = c8 + 8 * (tok >> 4);
      if (col >= cc) col -= cc;
      if (col >= cc) col -= cc;
      const float4 s0 = *reinterpret_cast<const float4*>(sS + tok * cc + col), s1 = *reinterpret_cast<const float4*>(sS + tok * cc + col + 4);
      const float S[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
      float y[8];
      Vec16<B>::load(static_cast<const B*>(a.y) + n * a.ldy + c, y);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float z = y[j] + a.y_bias[c + j];
        // z (1 + tanh(w)) / 2 = z / (1 + exp(-2 w))
        const float w2 = 1.5957691216057308f * fmaf(0.044715f * z * z, z, z);
        y[j] = a.scale * S[j] * z * fast_sigmoid(w2);
      }
      *reinterpret_cast<uint4*>(static_cast<B*>(a.out) + n * a.ldo + c) =
          make_uint4(pack_bf16x2(y[0], y[1]), pack_bf16x2(y[2], y[3]), pack_bf16x2(y[4], y[5]), pack_bf16x2(y[6], y[7]));
    }
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
  constexpr int kAhead = 16;
  for (int i0 = 0; i0 < n; i0 += kAhead) {
    float2 v[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j) v[j] = totals[(tile + min(i0 + j, n - 1)) * a.W + c];
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      if (i0 + j >= n) break;
      starts[(tile + i0 + j) * a.W + c] = S;
      S = fmaf(v[j].x, S, v[j].y);
    }
  }
  *sp = S;
}

bool lru_chunks_ok(const LruArgs& a) {
  const int wb = a.W / a.blocks;
  return wb % 16 == 0 && wb <= 512 && a.taps <= 8 && ((a.ldx | a.ldy | a.ldo) & 7) == 0 &&
         ((reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.out) |
           reinterpret_cast<uintptr_t>(a.gates) | reinterpret_cast<uintptr_t>(a.ring)) & 15) == 0;
}

// scratch: totals [tiles, W] float2, then starts [tiles, W], with tiles = n_tok / 64 + n_seq
cudaError_t lru_chunks_go(const SeqBatch& sb, const LruArgs& a, float* scratch, cudaStream_t st) {
  const int wb = a.W / a.blocks, tiles = sb.n_tok / kChunk + sb.n_seq, threads = min(wb, kSlice) * 2;
  const int rows = (2 + a.taps) * wb * 4, u = 2 * kChunk * staged_ld(wb) * 2, smem_u = u + rows, smem = u + max(rows, kChunk * min(wb, kSlice) * 4);
  static int have0 = 0, have1 = 0;
  cudaError_t e = want_smem(lru_chunk_kernel<false>, smem_u, have0);
  if (e == cudaSuccess) e = want_smem(lru_chunk_kernel<true>, smem, have1);
  if (e != cudaSuccess) return e;
  float2* totals = reinterpret_cast<float2*>(scratch);
  float* starts = scratch + static_cast<int64_t>(tiles) * a.W * 2;
  const dim3 grid(tiles, a.blocks, (wb + kSlice - 1) / kSlice);
  lru_chunk_kernel<false><<<grid, threads, smem_u, st>>>(sb, a, totals, nullptr);
  lru_prefix_kernel<<<dim3((a.W + 63) / 64, sb.n_seq), 64, 0, st>>>(sb, a, totals, starts);
  lru_chunk_kernel<true><<<grid, threads, smem, st>>>(sb, a, nullptr, starts);
  return lru_ring_go<__nv_bfloat16>(sb, a, st);
}

template <typename T>
cudaError_t lru_t(const SeqBatch& sb, const LruArgs& a, float* scratch, cudaStream_t st) {
  if (scratch == nullptr) return lru_gates_go<T, true>(sb, a, nullptr, nullptr, st);
  if constexpr (sizeof(T) == 2) {
    if (lru_chunks_ok(a)) return lru_chunks_go(sb, a, scratch, st);
  }
  float *log_a = scratch, *inp = scratch + static_cast<int64_t>(sb.n_tok) * a.W;
  const cudaError_t e = lru_gates_go<T, false>(sb, a, log_a, inp, st);
  if (e != cudaSuccess) return e;
  lru_scan_kernel<T><<<dim3((a.W + 63) / 64, sb.n_seq), 64, 0, st>>>(sb, a, log_a, inp);
  return lru_ring_go<T>(sb, a, st);
}

}  // namespace

int64_t gated_lru_scratch(bool f32, const SeqBatch& sb, const LruArgs& a) {
  const int64_t tiles = sb.n_tok / kChunk + sb.n_seq;
  return !f32 && lru_chunks_ok(a) ? 3 * tiles * a.W : 2 * static_cast<int64_t>(sb.n_tok) * a.W;
}

cudaError_t launch_gated_lru(bool f32, const SeqBatch& sb, const LruArgs& a, float* scratch, cudaStream_t st) {
  if (a.blocks < 1 || a.W % a.blocks != 0 || a.taps < 1 || (scratch == nullptr && sb.n_tok != sb.n_seq)) return cudaErrorInvalidValue;
  return f32 ? lru_t<float>(sb, a, scratch, st) : lru_t<__nv_bfloat16>(sb, a, scratch, st);
}

}  // namespace b200
