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

template <typename T>
cudaError_t lru_t(const SeqBatch& sb, const LruArgs& a, float* log_a, float* inp, cudaStream_t st) {
  if (log_a == nullptr) return lru_gates_go<T, true>(sb, a, nullptr, nullptr, st);
  const cudaError_t e = lru_gates_go<T, false>(sb, a, log_a, inp, st);
  if (e != cudaSuccess) return e;
  lru_scan_kernel<T><<<dim3((a.W + 63) / 64, sb.n_seq), 64, 0, st>>>(sb, a, log_a, inp);
  return lru_ring_go<T>(sb, a, st);
}

}  // namespace

cudaError_t launch_gated_lru(bool f32, const SeqBatch& sb, const LruArgs& a, float* log_a, float* inp, cudaStream_t st) {
  if (a.blocks < 1 || a.W % a.blocks != 0 || a.taps < 1 || (log_a == nullptr && sb.n_tok != sb.n_seq)) return cudaErrorInvalidValue;
  return f32 ? lru_t<float>(sb, a, log_a, inp, st) : lru_t<__nv_bfloat16>(sb, a, log_a, inp, st);
}

}  // namespace b200
