// Residual with several parallel streams on packed rows, and row-wise polynomial activations.
//
// stream_norm does what lies between two sublayers in one pass over the fp32 streams xs [rows, S, D]:
//   x_t <- sum_s mix[s, t] x_s + w_out[t] (y + bias)      (mix null: the sum is dropped, the streams start here)
//   u    = sum_s w_in[s] x_s
//   h    = u / rms(u) per group of D / groups features, times gamma
// poly_norm: a N(z) + b N(z^2) + c N(z^3) + e with N(v) = v / sqrt(mean(v^2) + eps) over the row.
//
// Sums, norms and powers are fp32. This file is built without fast-math.
#include "serve_common.cuh"
#include "serve_kernels.cuh"

namespace b200 {

namespace {

// ---- streams, any sizes: a block per row ----------------------------------------------------------------------------
template <typename TY, typename TO>
__global__ void stream_norm_kernel(const TY* __restrict__ y, const StreamNorm a, TO* __restrict__ h) {
  extern __shared__ float buf[];   // [D]
  const int64_t row = blockIdx.x;
  const int D = a.D, S = a.S;
  float* xr = a.xs + row * S * D;
  for (int i = threadIdx.x; i < D; i += blockDim.x) {
    float old[kMaxStreams];
    if (a.mix != nullptr)
      for (int s = 0; s < S; ++s) old[s] = xr[s * D + i];
    const float v = ldf(y + row * D + i) + (a.bias != nullptr ? a.bias[i] : 0.f);
    float u = 0.f;
    for (int t = 0; t < S; ++t) {
      float x = 0.f;
      if (a.mix != nullptr)
        for (int s = 0; s < S; ++s) x = fmaf(a.mix[s * S + t], old[s], x);
      x = fmaf(a.w_out[t], v, x);
      xr[t * D + i] = x;
      u = fmaf(a.w_in[t], x, u);
    }
    buf[i] = u;
    if (a.u != nullptr) a.u[row * D + i] = u;
  }
  if (h == nullptr) return;
  __syncthreads();
  const int size = D / a.groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  for (int g = warp; g < a.groups; g += nw) {
    float q = 0.f;
    for (int i = lane; i < size; i += 32) q += buf[g * size + i] * buf[g * size + i];
    const float inv = 1.f / sqrtf(warp_sum(q) / size + a.eps);
    for (int i = lane; i < size; i += 32) stf(h + row * D + g * size + i, buf[g * size + i] * inv * a.gamma[g * size + i]);
  }
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
__device__ __forceinline__ float4 fma4(float w, const float4& a, const float4& c) {
  return make_float4(fmaf(w, a.x, c.x), fmaf(w, a.y, c.y), fmaf(w, a.z, c.z), fmaf(w, a.w, c.w));
}

// Four features per thread and step, u in registers. Groups are multiples of 128 features (a warp's step lies in one) or
// powers of two below (some lanes of a warp's step).
template <typename TY, typename TO, int S, int kIt, int kThr>
__global__ void __launch_bounds__(kThr)
stream_norm_vec_kernel(const TY* __restrict__ y, const StreamNorm a, TO* __restrict__ h) {
  __shared__ float seg[kIt * kThr / 32];
  const int64_t row = blockIdx.x;
  const int D = a.D, t = threadIdx.x, size = D / a.groups;
  float* xr = a.xs + row * S * D;
  float mix[S][S], wo[S], wi[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    wi[s] = a.w_in[s];
    wo[s] = a.w_out[s];
#pragma unroll
    for (int p = 0; p < S; ++p) mix[s][p] = a.mix != nullptr ? a.mix[s * S + p] : 0.f;
  }
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 u[kIt];
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + t) * 4;
    u[k] = zero;
    if (i < D) {
      float4 x[S];
#pragma unroll
      for (int s = 0; s < S; ++s) x[s] = a.mix != nullptr ? *reinterpret_cast<const float4*>(xr + s * D + i) : zero;
      float4 v = ld4(y + row * D + i);
      if (a.bias != nullptr) {
        const float4 b = *reinterpret_cast<const float4*>(a.bias + i);
        v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
      }
#pragma unroll
      for (int p = 0; p < S; ++p) {
        float4 n = zero;
#pragma unroll
        for (int s = 0; s < S; ++s) n = fma4(mix[s][p], x[s], n);
        n = fma4(wo[p], v, n);
        *reinterpret_cast<float4*>(xr + p * D + i) = n;
        u[k] = fma4(wi[p], n, u[k]);
      }
      if (a.u != nullptr) *reinterpret_cast<float4*>(a.u + row * D + i) = u[k];
    }
  }
  if (h == nullptr) return;
  float q[kIt];
#pragma unroll
  for (int k = 0; k < kIt; ++k) q[k] = (u[k].x * u[k].x + u[k].y * u[k].y) + (u[k].z * u[k].z + u[k].w * u[k].w);
  if (size >= 128) {
#pragma unroll
    for (int k = 0; k < kIt; ++k) {
      const float w = warp_sum(q[k]);
      if ((t & 31) == 0) seg[(k * kThr + t) >> 5] = w;
    }
    __syncthreads();
    const int per = size >> 7;
    int have = -1;
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < kIt; ++k) {
      const int i = (k * kThr + t) * 4, g = i / size;
      if (i < D && g != have) {
        have = g;
        sum = 0.f;
        for (int p = 0; p < per; ++p) sum += seg[g * per + p];
      }
      q[k] = sum;
    }
  } else {
#pragma unroll
    for (int k = 0; k < kIt; ++k)
      for (int o = size >> 3; o > 0; o >>= 1) q[k] += __shfl_xor_sync(0xffffffffu, q[k], o);
  }
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + t) * 4;
    if (i < D) {
      const float inv = 1.f / sqrtf(q[k] / size + a.eps);
      const float4 g = *reinterpret_cast<const float4*>(a.gamma + i);
      const float4 r = make_float4(u[k].x * inv * g.x, u[k].y * inv * g.y, u[k].z * inv * g.z, u[k].w * inv * g.w);
      if constexpr (sizeof(TO) == 2) *reinterpret_cast<uint2*>(h + row * D + i) = make_uint2(pack_bf16x2(r.x, r.y), pack_bf16x2(r.z, r.w));
      else *reinterpret_cast<float4*>(h + row * D + i) = r;
    }
  }
}

template <typename TY, typename TO, int S>
bool stream_norm_vec(const TY* y, const StreamNorm& a, TO* h, cudaStream_t st) {
  const int D = a.D, size = D / a.groups;
  const bool groups_ok = size % 128 == 0 || (size >= 4 && size < 128 && (size & (size - 1)) == 0);
  if (D % 4 != 0 || D > 16384 || (h != nullptr && !groups_ok) ||
      ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(a.xs) | reinterpret_cast<uintptr_t>(a.bias) |
        reinterpret_cast<uintptr_t>(a.gamma) | reinterpret_cast<uintptr_t>(a.u) | reinterpret_cast<uintptr_t>(h)) & 15) != 0)
    return false;
#define B200_SN(IT, THR) stream_norm_vec_kernel<TY, TO, S, IT, THR><<<a.rows, THR, 0, st>>>(y, a, h)
  if (D <= 512) B200_SN(1, 128);
  else if (D <= 1024) B200_SN(1, 256);
  else if (D <= 2048) B200_SN(2, 256);
  else if (D <= 4096) B200_SN(2, 512);
  else if (D <= 8192) B200_SN(4, 512);
  else B200_SN(8, 512);
#undef B200_SN
  return true;
}

template <typename TY, typename TO>
cudaError_t stream_norm_t(const TY* y, const StreamNorm& a, TO* h, cudaStream_t st) {
  bool done = false;
  if (a.S == 1) done = stream_norm_vec<TY, TO, 1>(y, a, h, st);
  else if (a.S == 2) done = stream_norm_vec<TY, TO, 2>(y, a, h, st);
  else if (a.S == 3) done = stream_norm_vec<TY, TO, 3>(y, a, h, st);
  else if (a.S == 4) done = stream_norm_vec<TY, TO, 4>(y, a, h, st);
  if (!done) {
    static int have = 0;
    const cudaError_t e = want_smem(stream_norm_kernel<TY, TO>, a.D * 4, have);
    if (e != cudaSuccess) return e;
    stream_norm_kernel<TY, TO><<<a.rows, a.D >= 1024 ? 256 : 128, a.D * 4, st>>>(y, a, h);
  }
  return cudaGetLastError();
}

// ---- polynomial of normalised powers --------------------------------------------------------------------------------
struct PolySums {
  float s2, s4, s6;
  __device__ __forceinline__ void add(float z) {
    const float q = z * z, c = q * z;
    s2 += q;
    s4 = fmaf(q, q, s4);
    s6 = fmaf(c, c, s6);
  }
};
struct PolyScale {
  float a, b, c, e;   // value = a z + b z^2 + c z^3 + e with the norms folded in
  __device__ __forceinline__ float at(float z) const { return fmaf(z, fmaf(z, fmaf(z, c, b), a), e); }
};
// The block's sums -> factors of this row; red holds 3 * 32 + 4 floats.
__device__ __forceinline__ PolyScale poly_scale(const PolySums& p, const float* coef, int N, float eps, float* red) {
  const float v2 = warp_sum(p.s2), v4 = warp_sum(p.s4), v6 = warp_sum(p.s6);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) {
    red[warp] = v2;
    red[32 + warp] = v4;
    red[64 + warp] = v6;
  }
  __syncthreads();
  if (warp < 3) {
    const float v = warp_sum(lane < nw ? red[warp * 32 + lane] : 0.f);
    if (lane == 0) red[96 + warp] = coef[warp] / sqrtf(v / N + eps);
  }
  __syncthreads();
  return PolyScale{red[96], red[97], red[98], coef[3]};
}

template <typename T>
__global__ void poly_norm_kernel(const T* __restrict__ z, int64_t ldz, const float* __restrict__ coef, T* __restrict__ out, int N, float eps) {
  __shared__ float red[100];
  const T* zr = z + static_cast<int64_t>(blockIdx.x) * ldz;
  T* o = out + static_cast<int64_t>(blockIdx.x) * N;
  PolySums p{0.f, 0.f, 0.f};
  for (int i = threadIdx.x; i < N; i += blockDim.x) p.add(ldf(zr + i));
  const PolyScale s = poly_scale(p, coef, N, eps, red);
  for (int i = threadIdx.x; i < N; i += blockDim.x) stf(o + i, s.at(ldf(zr + i)));
}

// bf16, eight features per thread and step, the row in registers.
template <int kIt, int kThr>
__global__ void __launch_bounds__(kThr)
poly_norm_vec_kernel(const __nv_bfloat16* __restrict__ z, int64_t ldz, const float* __restrict__ coef, __nv_bfloat16* __restrict__ out,
                     int N, float eps) {
  __shared__ float red[100];
  const __nv_bfloat16* zr = z + static_cast<int64_t>(blockIdx.x) * ldz;
  __nv_bfloat16* o = out + static_cast<int64_t>(blockIdx.x) * N;
  uint4 v[kIt];
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + threadIdx.x) * 8;
    v[k] = i < N ? *reinterpret_cast<const uint4*>(zr + i) : make_uint4(0u, 0u, 0u, 0u);
  }
  PolySums p{0.f, 0.f, 0.f};
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const uint32_t w[4] = {v[k].x, v[k].y, v[k].z, v[k].w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = unpack_bf16x2(w[j]);
      p.add(f.x);
      p.add(f.y);
    }
  }
  const PolyScale s = poly_scale(p, coef, N, eps, red);
#pragma unroll
  for (int k = 0; k < kIt; ++k) {
    const int i = (k * kThr + threadIdx.x) * 8;
    uint32_t w[4] = {v[k].x, v[k].y, v[k].z, v[k].w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = unpack_bf16x2(w[j]);
      w[j] = pack_bf16x2(s.at(f.x), s.at(f.y));
    }
    if (i < N) *reinterpret_cast<uint4*>(o + i) = make_uint4(w[0], w[1], w[2], w[3]);
  }
}

}  // namespace

cudaError_t launch_stream_norm(bool y_f32, bool f32_out, const void* y, const StreamNorm& a, void* h, cudaStream_t st) {
  if (a.S < 1 || a.S > kMaxStreams || a.groups < 1 || a.D % a.groups != 0 || (h != nullptr && a.gamma == nullptr) || (!y_f32 && f32_out))
    return cudaErrorInvalidValue;
  using B = __nv_bfloat16;
  if (f32_out) return stream_norm_t<float, float>(static_cast<const float*>(y), a, static_cast<float*>(h), st);
  if (y_f32) return stream_norm_t<float, B>(static_cast<const float*>(y), a, static_cast<B*>(h), st);
  return stream_norm_t<B, B>(static_cast<const B*>(y), a, static_cast<B*>(h), st);
}

cudaError_t launch_poly_norm(bool f32, const void* z, int64_t ldz, const float* coef, void* out, int rows, int N, float eps, cudaStream_t st) {
  if (f32) {
    poly_norm_kernel<float><<<rows, N >= 1024 ? 512 : 128, 0, st>>>(static_cast<const float*>(z), ldz, coef, static_cast<float*>(out), N, eps);
    return cudaGetLastError();
  }
  const __nv_bfloat16* zb = static_cast<const __nv_bfloat16*>(z);
  __nv_bfloat16* o = static_cast<__nv_bfloat16*>(out);
  const bool vec = N % 8 == 0 && ldz % 8 == 0 && ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
#define B200_PN(IT, THR) poly_norm_vec_kernel<IT, THR><<<rows, THR, 0, st>>>(zb, ldz, coef, o, N, eps)
  if (vec && N <= 1024) B200_PN(1, 128);
  else if (vec && N <= 2048) B200_PN(1, 256);
  else if (vec && N <= 4096) B200_PN(2, 256);
  else if (vec && N <= 8192) B200_PN(4, 256);
  else if (vec && N <= 16384) B200_PN(4, 512);
  else if (vec && N <= 32768) B200_PN(8, 512);
  else poly_norm_kernel<__nv_bfloat16><<<rows, N >= 1024 ? 512 : 128, 0, st>>>(zb, ldz, coef, o, N, eps);
#undef B200_PN
  return cudaGetLastError();
}

}  // namespace b200
