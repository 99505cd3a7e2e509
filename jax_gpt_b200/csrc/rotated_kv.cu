// Attention operands with interleaved rotary pairs (2i, 2i + 1) and rotated values, on packed batches.
//
// qkv_rotate: a projection row holds q (H heads of dk), k (G of dk) and v (G of dv) at given columns. With the biases added, q
// and k turn by the tables of `rope` (their first rope.dims features, amplitude folded in), v by the tables of `vrope`
// over all dv features. The cache row [K of every kv head | V of every kv head] is written, q goes to [n_tok, H, dkp], and for
// whole prompts k and v also to dense operands [n_tok, G, dkp], [n_tok, G, dvp]; features past dk / dv are zero there, so that a
// tensor-core kernel of the next larger width takes heads of any size.
//
// turn_back_gate: the output of a head at position i is the sum of values turned by their own positions; turning it by -i leaves
// values turned by relative positions. It is then multiplied by sigmoid(g) of the head and by a constant.
//
// Angles, turns and gates are fp32. This file is built without fast-math.
#include "serve_common.cuh"
#include "serve_kernels.cuh"

namespace b200 {

namespace {

struct RotArgs {
  SeqBatch sb;
  QkvRows in;
  RopeTable rope, vrope;
  PagedRows pages;
  int H, G, dk, dv, dkp, dvp;
  int* status;
};

// where a padded feature of a token comes from and goes to: 0 q, 1 k, 2 v
struct Feature {
  int kind, head, c;
};

__device__ __forceinline__ Feature feature_of(const RotArgs& a, int i) {
  const int nq = a.H * a.dkp, nk = a.G * a.dkp;
  if (i < nq) return {0, i / a.dkp, i % a.dkp};
  if (i < nq + nk) return {1, (i - nq) / a.dkp, (i - nq) % a.dkp};
  return {2, (i - nq - nk) / a.dvp, (i - nq - nk) % a.dvp};
}

template <typename T>
__global__ void __launch_bounds__(256)
qkv_rotate_kernel(const RotArgs a, T* __restrict__ qo, T* __restrict__ ko, T* __restrict__ vo) {
  const int n = blockIdx.x, b = a.sb.tok_seq[n], pos = a.sb.start[b] + n - a.sb.cu[b];
  const int64_t dst = page_row(a.pages, a.sb.ids[b], pos);
  if (dst < 0 || pos >= a.rope.max_pos || pos >= a.vrope.max_pos) {
    if (threadIdx.x == 0) report_status(a.status, kBadArgument, 340, b, pos);
    return;
  }
  const T* row = static_cast<const T*>(a.in.y) + static_cast<int64_t>(n) * a.in.ld;
  T* cache = static_cast<T*>(a.pages.pool) + dst * a.pages.width;
  const int total = (a.H + a.G) * a.dkp + a.G * a.dvp;
  for (int i = threadIdx.x; i < total; i += blockDim.x) {
    const Feature f = feature_of(a, i);
    const int d = f.kind == 2 ? a.dv : a.dk, col = f.kind == 0 ? a.in.q : f.kind == 1 ? a.in.k : a.in.v;
    const float* bias = f.kind == 0 ? a.in.bq : f.kind == 1 ? a.in.bk : a.in.bv;
    const RopeTable& r = f.kind == 2 ? a.vrope : a.rope;
    auto at = [&](int c) { return ldf(row + col + f.head * d + c) + (bias != nullptr ? bias[f.head * d + c] : 0.f); };
    float v = 0.f;
    if (f.c < r.dims) {
      const int64_t k = static_cast<int64_t>(pos) * (r.dims / 2) + (f.c >> 1);
      const float cs = r.cos[k], sn = r.sin[k];
      v = (f.c & 1) == 0 ? at(f.c) * cs - at(f.c + 1) * sn : at(f.c) * cs + at(f.c - 1) * sn;
    } else if (f.c < d) {
      v = at(f.c);
    }
    if (f.kind == 0) {
      stf(qo + (static_cast<int64_t>(n) * a.H + f.head) * a.dkp + f.c, v);
    } else {
      if (f.c < d) stf(cache + (f.kind == 1 ? 0 : a.G * a.dk) + f.head * d + f.c, v);
      if (f.kind == 1 && ko != nullptr) stf(ko + (static_cast<int64_t>(n) * a.G + f.head) * a.dkp + f.c, v);
      if (f.kind == 2 && vo != nullptr) stf(vo + (static_cast<int64_t>(n) * a.G + f.head) * a.dvp + f.c, v);
    }
  }
}

// eight features = four pairs turned by cos[0..3], sin[0..3]
__device__ __forceinline__ void turn8(float (&f)[8], const float* cos, const float* sin, float dir) {
  const float4 c4 = *reinterpret_cast<const float4*>(cos), s4 = *reinterpret_cast<const float4*>(sin);
  const float c[4] = {c4.x, c4.y, c4.z, c4.w}, s[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float u = f[2 * j], v = f[2 * j + 1], w = dir * s[j];
    f[2 * j] = u * c[j] - v * w;
    f[2 * j + 1] = v * c[j] + u * w;
  }
}
__device__ __forceinline__ uint4 pack8(const float (&f)[8], float w = 1.f) {
  return make_uint4(pack_bf16x2(f[0] * w, f[1] * w), pack_bf16x2(f[2] * w, f[3] * w), pack_bf16x2(f[4] * w, f[5] * w),
                    pack_bf16x2(f[6] * w, f[7] * w));
}

// bf16 with every width, column and rotated width a multiple of 8: eight features per thread and step.
__global__ void __launch_bounds__(256)
qkv_rotate_vec_kernel(const RotArgs a, __nv_bfloat16* __restrict__ qo, __nv_bfloat16* __restrict__ ko, __nv_bfloat16* __restrict__ vo) {
  using B = __nv_bfloat16;
  const int n = blockIdx.x, b = a.sb.tok_seq[n], pos = a.sb.start[b] + n - a.sb.cu[b];
  const int64_t dst = page_row(a.pages, a.sb.ids[b], pos);
  if (dst < 0 || pos >= a.rope.max_pos || pos >= a.vrope.max_pos) {
    if (threadIdx.x == 0) report_status(a.status, kBadArgument, 340, b, pos);
    return;
  }
  const B* row = static_cast<const B*>(a.in.y) + static_cast<int64_t>(n) * a.in.ld;
  B* cache = static_cast<B*>(a.pages.pool) + dst * a.pages.width;
  const int total = ((a.H + a.G) * a.dkp + a.G * a.dvp) / 8;
  for (int i = threadIdx.x; i < total; i += blockDim.x) {
    const Feature f = feature_of(a, i * 8);
    const int d = f.kind == 2 ? a.dv : a.dk;
    uint4 out = make_uint4(0u, 0u, 0u, 0u);
    if (f.c < d) {
      const int col = f.kind == 0 ? a.in.q : f.kind == 1 ? a.in.k : a.in.v;
      const float* bias = f.kind == 0 ? a.in.bq : f.kind == 1 ? a.in.bk : a.in.bv;
      const RopeTable& r = f.kind == 2 ? a.vrope : a.rope;
      float v[8];
      Vec16<B>::load(row + col + f.head * d + f.c, v);
      if (bias != nullptr) {
        const float4 x = *reinterpret_cast<const float4*>(bias + f.head * d + f.c), z = *reinterpret_cast<const float4*>(bias + f.head * d + f.c + 4);
        v[0] += x.x; v[1] += x.y; v[2] += x.z; v[3] += x.w;
        v[4] += z.x; v[5] += z.y; v[6] += z.z; v[7] += z.w;
      }
      if (f.c < r.dims) {
        const int64_t k = static_cast<int64_t>(pos) * (r.dims / 2) + (f.c >> 1);
        turn8(v, r.cos + k, r.sin + k, 1.f);
      }
      out = pack8(v);
    }
    if (f.kind == 0) {
      *reinterpret_cast<uint4*>(qo + (static_cast<int64_t>(n) * a.H + f.head) * a.dkp + f.c) = out;
    } else {
      if (f.c < d) *reinterpret_cast<uint4*>(cache + (f.kind == 1 ? 0 : a.G * a.dk) + f.head * d + f.c) = out;
      if (f.kind == 1 && ko != nullptr) *reinterpret_cast<uint4*>(ko + (static_cast<int64_t>(n) * a.G + f.head) * a.dkp + f.c) = out;
      if (f.kind == 2 && vo != nullptr) *reinterpret_cast<uint4*>(vo + (static_cast<int64_t>(n) * a.G + f.head) * a.dvp + f.c) = out;
    }
  }
}

template <typename T, bool kVec>
__global__ void __launch_bounds__(256)
turn_back_gate_kernel(const SeqBatch sb, const T* __restrict__ o, int ldh, const T* __restrict__ g, int64_t ldg, const RopeTable vrope, float scale,
                      int H, int dv, T* __restrict__ out, int64_t ldo) {
  const int n = blockIdx.x, b = sb.tok_seq[n], pos = min(sb.start[b] + n - sb.cu[b], vrope.max_pos - 1);
  const T* src = o + static_cast<int64_t>(n) * H * ldh;
  T* dst = out + static_cast<int64_t>(n) * ldo;
  const int half = vrope.dims / 2;
  const float* cs = vrope.cos + static_cast<int64_t>(pos) * half;
  const float* sn = vrope.sin + static_cast<int64_t>(pos) * half;
  if constexpr (kVec) {
    for (int i = threadIdx.x; i < H * dv / 8; i += blockDim.x) {
      const int h = i * 8 / dv, c = i * 8 % dv;
      float v[8];
      Vec16<T>::load(src + h * ldh + c, v);
      if (c < vrope.dims) turn8(v, cs + (c >> 1), sn + (c >> 1), -1.f);
      *reinterpret_cast<uint4*>(dst + h * dv + c) = pack8(v, scale * sigmoid_f(ldf(g + n * ldg + h)));
    }
  } else {
    for (int i = threadIdx.x; i < H * dv; i += blockDim.x) {
      const int h = i / dv, c = i % dv;
      const T* p = src + h * ldh;
      float v = ldf(p + c);
      if (c < vrope.dims) {
        const float x = cs[c >> 1], s = sn[c >> 1];
        v = (c & 1) == 0 ? v * x + ldf(p + c + 1) * s : v * x - ldf(p + c - 1) * s;
      }
      stf(dst + i, v * (scale * sigmoid_f(ldf(g + n * ldg + h))));
    }
  }
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

cudaError_t launch_qkv_rotate(bool f32, const SeqBatch& sb, const QkvRows& in, const RopeTable& rope, const RopeTable& vrope,
                              const PagedRows& pages, int H, int G, int dk, int dv, int dkp, int dvp, void* q, void* k, void* v, int* status,
                              cudaStream_t st) {
  if (pages.width != G * (dk + dv) || rope.dims > dk || vrope.dims > dv || dkp < dk || dvp < dv) return cudaErrorInvalidValue;
  const RotArgs a{sb, in, rope, vrope, pages, H, G, dk, dv, dkp, dvp, status};
  if (f32) {
    qkv_rotate_kernel<float><<<sb.n_tok, 256, 0, st>>>(a, static_cast<float*>(q), static_cast<float*>(k), static_cast<float*>(v));
    return cudaGetLastError();
  }
  using B = __nv_bfloat16;
  B *qb = static_cast<B*>(q), *kb = static_cast<B*>(k), *vb = static_cast<B*>(v);
  const bool vec = ((dk | dv | dkp | dvp | rope.dims | vrope.dims | in.q | in.k | in.v | in.ld) & 7) == 0 && aligned16(in.y) && aligned16(in.bq) &&
                   aligned16(in.bk) && aligned16(in.bv) && aligned16(rope.cos) && aligned16(rope.sin) && aligned16(vrope.cos) && aligned16(vrope.sin);
  if (vec) {
    const int units = ((H + G) * dkp + G * dvp) / 8;
    qkv_rotate_vec_kernel<<<sb.n_tok, units <= 64 ? 64 : units <= 128 ? 128 : 256, 0, st>>>(a, qb, kb, vb);
  } else {
    qkv_rotate_kernel<B><<<sb.n_tok, 256, 0, st>>>(a, qb, kb, vb);
  }
  return cudaGetLastError();
}

cudaError_t launch_turn_back_gate(bool f32, const SeqBatch& sb, const void* o, int ldh, const void* g, int64_t ldg, const RopeTable& vrope,
                                  float scale, int H, int dv, void* out, int64_t ldo, cudaStream_t st) {
  if (vrope.dims > dv || ldh < dv) return cudaErrorInvalidValue;
  if (f32) {
    turn_back_gate_kernel<float, false><<<sb.n_tok, 256, 0, st>>>(sb, static_cast<const float*>(o), ldh, static_cast<const float*>(g), ldg, vrope,
                                                                  scale, H, dv, static_cast<float*>(out), ldo);
    return cudaGetLastError();
  }
  using B = __nv_bfloat16;
  const B *ob = static_cast<const B*>(o), *gb = static_cast<const B*>(g);
  B* d = static_cast<B*>(out);
  const bool vec = ((dv | ldh | vrope.dims | ldo) & 7) == 0 && aligned16(o) && aligned16(out) && aligned16(vrope.cos) && aligned16(vrope.sin);
  const int units = H * dv / 8;
  if (vec) turn_back_gate_kernel<B, true><<<sb.n_tok, units <= 64 ? 64 : units <= 128 ? 128 : 256, 0, st>>>(sb, ob, ldh, gb, ldg, vrope, scale, H, dv, d, ldo);
  else turn_back_gate_kernel<B, false><<<sb.n_tok, 256, 0, st>>>(sb, ob, ldh, gb, ldg, vrope, scale, H, dv, d, ldo);
  return cudaGetLastError();
}

}  // namespace b200
