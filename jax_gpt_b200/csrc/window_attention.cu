// Grouped-query attention with a sliding window and kept first tokens on packed batches over paged key / value rows:
//   position i sees j when j <= i and (i - j < size or j < keep_first),
// or instead of the first tokens one mean key and value for every block of tokens that lies wholly before the window. Scores may be
// soft-capped, the denominator may hold a sink.
//
// qk_prepare turns a projection row [q heads | k heads] into attention operands (bias, half-split rotation, unit RMS norm
// per head) and writes the cache row [K of every kv head | V of every kv head]; the projected keys double as values.
// window_attention is the attention for any sizes, fp32 or bf16, prompts that continue a cache and decode steps with split
// keys; it walks only the key tiles that some query of the block can see. The tensor-core forms are in attention_sm100.cu
// (whole prompts) and attention_decode.cu (one token).
//
// Angles, norms, scores and softmax are fp32. This file is built without fast-math.
#include "serve_common.cuh"
#include "serve_kernels.cuh"

namespace b200 {

namespace {

// ---- operands ------------------------------------------------------------------------------------------------------------
struct PrepArgs {
  SeqBatch sb;
  const float* bias;      // [(H + G) * D] or null
  int H, G, D;
  float eps;
  int unit_norm;
  RopeTable rope;         // half-split pairs (i, i + dims / 2)
  PagedRows pages;
  int64_t ldy;
  int* status;
};

// A warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256)
qk_prepare_kernel(const PrepArgs a, const T* __restrict__ y, T* __restrict__ qo, T* __restrict__ ko, T* __restrict__ vo) {
  const int heads = a.H + a.G, D = a.D, half = a.rope.dims / 2;
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (unit >= static_cast<int64_t>(a.sb.n_tok) * heads) return;
  const int n = static_cast<int>(unit / heads), h = static_cast<int>(unit % heads), lane = threadIdx.x & 31;
  const int b = a.sb.tok_seq[n], pos = a.sb.start[b] + n - a.sb.cu[b];
  const int64_t dst = page_row(a.pages, a.sb.ids[b], pos);
  if (dst < 0 || pos >= a.rope.max_pos) {
    if (lane == 0) report_status(a.status, kBadArgument, 330, b, pos);
    return;
  }
  const T* row = y + static_cast<int64_t>(n) * a.ldy + h * D;
  const float* bias = a.bias != nullptr ? a.bias + h * D : nullptr;
  auto at = [&](int i) { return ldf(row + i) + (bias != nullptr ? bias[i] : 0.f); };
  const float* cs = a.rope.cos + static_cast<int64_t>(pos) * half;
  const float* sn = a.rope.sin + static_cast<int64_t>(pos) * half;
  auto turned = [&](int i) {
    if (i < half) return at(i) * cs[i] - at(i + half) * sn[i];
    if (i < 2 * half) return at(i) * cs[i - half] + at(i - half) * sn[i - half];
    return at(i);
  };
  float s = 0.f;
  for (int i = lane; i < D; i += 32) { const float v = turned(i); s += v * v; }
  const float inv = a.unit_norm ? 1.f / sqrtf(warp_sum(s) / D + a.eps) : 1.f;
  if (h < a.H) {
    T* q = qo + static_cast<int64_t>(n) * a.H * D + h * D;
    for (int i = lane; i < D; i += 32) stf(q + i, turned(i) * inv);
    return;
  }
  const int g = h - a.H;
  T* ck = static_cast<T*>(a.pages.pool) + dst * a.pages.width + g * D;
  T* cv = ck + a.G * D;
  const int64_t dense = (static_cast<int64_t>(n) * a.G + g) * D;
  for (int i = lane; i < D; i += 32) {
    const float k = turned(i) * inv, v = at(i);
    stf(ck + i, k);
    stf(cv + i, v);
    if (ko != nullptr) {
      stf(ko + dense + i, k);
      stf(vo + dense + i, v);
    }
  }
}

// bf16, D and the rotated width multiples of 16: L lanes per (token, head), each with two chunks of eight features (a
// rotated pair of chunks, or two neighbours of the unrotated rest). D <= 16 * L.
template <int L>
__global__ void __launch_bounds__(256)
qk_prepare_vec_kernel(const PrepArgs a, const __nv_bfloat16* __restrict__ y, __nv_bfloat16* __restrict__ qo,
                      __nv_bfloat16* __restrict__ ko, __nv_bfloat16* __restrict__ vo) {
  using B = __nv_bfloat16;
  const int heads = a.H + a.G, D = a.D, half = a.rope.dims / 2;
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * (256 / L) + threadIdx.x / L;
  const bool live = unit < static_cast<int64_t>(a.sb.n_tok) * heads;
  const int n = live ? static_cast<int>(unit / heads) : 0, h = live ? static_cast<int>(unit % heads) : 0, p = threadIdx.x % L;
  const int b = a.sb.tok_seq[n], pos = a.sb.start[b] + n - a.sb.cu[b];
  const int64_t dst = page_row(a.pages, a.sb.ids[b], pos);
  const bool ok = live && dst >= 0 && pos < a.rope.max_pos;
  if (live && !ok && p == 0) report_status(a.status, kBadArgument, 330, b, pos);
  const bool rot = p < half / 8, in = ok && p < D / 16;
  const int c0 = rot ? 8 * p : 2 * half + 16 * (p - half / 8), c1 = rot ? half + 8 * p : c0 + 8;
  float u[8], v[8], ru[8], rv[8], s = 0.f;
  if (in) {
    const B* row = y + static_cast<int64_t>(n) * a.ldy + h * D;
    Vec16<B>::load(row + c0, u);
    Vec16<B>::load(row + c1, v);
    if (a.bias != nullptr) {
#pragma unroll
      for (int j = 0; j < 8; j += 4) {
        const float4 x = *reinterpret_cast<const float4*>(a.bias + h * D + c0 + j), z = *reinterpret_cast<const float4*>(a.bias + h * D + c1 + j);
        u[j] += x.x; u[j + 1] += x.y; u[j + 2] += x.z; u[j + 3] += x.w;
        v[j] += z.x; v[j + 1] += z.y; v[j + 2] += z.z; v[j + 3] += z.w;
      }
    }
    if (rot) {
      const float* cs = a.rope.cos + static_cast<int64_t>(pos) * half + 8 * p;
      const float* sn = a.rope.sin + static_cast<int64_t>(pos) * half + 8 * p;
#pragma unroll
      for (int j = 0; j < 8; j += 4) {
        const float4 c = *reinterpret_cast<const float4*>(cs + j), d = *reinterpret_cast<const float4*>(sn + j);
        const float ca[4] = {c.x, c.y, c.z, c.w}, sa[4] = {d.x, d.y, d.z, d.w};
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          ru[j + k] = u[j + k] * ca[k] - v[j + k] * sa[k];
          rv[j + k] = v[j + k] * ca[k] + u[j + k] * sa[k];
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) { ru[j] = u[j]; rv[j] = v[j]; }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) s += ru[j] * ru[j] + rv[j] * rv[j];
  }
#pragma unroll
  for (int o = L / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
  if (!in) return;
  const float inv = a.unit_norm ? 1.f / sqrtf(s / D + a.eps) : 1.f;
  auto pack = [](const float (&f)[8], float w) {
    return make_uint4(pack_bf16x2(f[0] * w, f[1] * w), pack_bf16x2(f[2] * w, f[3] * w), pack_bf16x2(f[4] * w, f[5] * w),
                      pack_bf16x2(f[6] * w, f[7] * w));
  };
  const uint4 w0 = pack(ru, inv), w1 = pack(rv, inv);
  if (h < a.H) {
    B* q = qo + static_cast<int64_t>(n) * a.H * D + h * D;
    *reinterpret_cast<uint4*>(q + c0) = w0;
    *reinterpret_cast<uint4*>(q + c1) = w1;
    return;
  }
  const int g = h - a.H;
  const uint4 x0 = pack(u, 1.f), x1 = pack(v, 1.f);
  B* ck = static_cast<B*>(a.pages.pool) + dst * a.pages.width + g * D;
  B* cv = ck + a.G * D;
  *reinterpret_cast<uint4*>(ck + c0) = w0;
  *reinterpret_cast<uint4*>(ck + c1) = w1;
  *reinterpret_cast<uint4*>(cv + c0) = x0;
  *reinterpret_cast<uint4*>(cv + c1) = x1;
  if (ko != nullptr) {
    const int64_t dense = (static_cast<int64_t>(n) * a.G + g) * D;
    *reinterpret_cast<uint4*>(ko + dense + c0) = w0;
    *reinterpret_cast<uint4*>(ko + dense + c1) = w1;
    *reinterpret_cast<uint4*>(vo + dense + c0) = x0;
    *reinterpret_cast<uint4*>(vo + dense + c1) = x1;
  }
}

// ---- attention, any sizes ------------------------------------------------------------------------------------------------
// The work items of a sequence and kv head are its (token, query head of the group) pairs with the head running fastest; a
// block owns kWaQ consecutive pairs and walks its visible keys in tiles of 32 staged in shared memory as fp32. Warp w
// scores pairs w and w + 4 with one key per lane and accumulates their outputs in shared memory.
constexpr int kWaQ = 8, kWaK = 32, kWaWarps = 4, kWaMine = kWaQ / kWaWarps;

template <typename T>
__device__ __forceinline__ void stage_row(const T* __restrict__ src, bool live, int n, int lane, float* dst) {
  if (live && n % Vec16<T>::n == 0 && (reinterpret_cast<uintptr_t>(src) & 15) == 0) {
    for (int i = lane * Vec16<T>::n; i < n; i += 32 * Vec16<T>::n) {
      float f[Vec16<T>::n];
      Vec16<T>::load(src + i, f);
#pragma unroll
      for (int j = 0; j < Vec16<T>::n; ++j) dst[i + j] = f[j];
    }
  } else {
    for (int i = lane; i < n; i += 32) dst[i] = live ? ldf(src + i) : 0.f;
  }
}

template <typename T>
__global__ void __launch_bounds__(kWaWarps * 32)
window_attn_kernel(const SeqBatch sb, const T* __restrict__ qx, const PagedRows pages, const T* __restrict__ pooled, int H, int G, int D, int DV,
                   WindowMask mask, const ScoreArgs score, float* __restrict__ part_o, float* __restrict__ part_ml, T* __restrict__ out) {
  extern __shared__ float sm[];
  const int DS = D | 1;                    // odd stride: lanes read a column of keys without bank conflicts
  float* sk = sm;                          // [kWaK][DS]
  float* sv = sk + kWaK * DS;              // [kWaK][DV]
  float* sq = sv + kWaK * DV;              // [kWaQ][D]
  float* so = sq + kWaQ * D;               // [kWaQ][DV]
  float* sp = so + kWaQ * DV;              // [kWaQ][kWaK]
  const int split = blockIdx.y, S = gridDim.y, g = blockIdx.z, rep = H / G;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int tile = blockIdx.x, b = 0, r0 = -1, cnt = 0;      // tile -> (sequence, first pair)
  for (; b < sb.n_seq; ++b) {
    const int pairs = (sb.cu[b + 1] - sb.cu[b]) * rep, tiles = (pairs + kWaQ - 1) / kWaQ;
    if (tile < tiles) {
      r0 = tile * kWaQ;
      cnt = min(kWaQ, pairs - r0);
      break;
    }
    tile -= tiles;
  }
  if (r0 < 0) return;
  const int slot = sb.ids[b], start = sb.start[b];
  const int p_lo = start + r0 / rep, p_hi = start + (r0 + cnt - 1) / rep;
  // visible key tiles: the kept first keys or the block means, then from the window of the first query to the last query
  const bool blocks = mask.pool > 0;
  const int kept = blocks ? blocks_seen(p_hi, mask.size, mask.pool) : min(mask.keep_first, p_hi + 1);
  const int n_keep = (kept + kWaK - 1) / kWaK;
  const int w0 = max(blocks ? 0 : n_keep, max(0, p_lo - mask.size + 1) / kWaK), w1 = p_hi / kWaK + 1;
  const int n_tiles = n_keep + max(0, w1 - w0), per = (n_tiles + S - 1) / S;
  const int i0 = split * per, i1 = min(n_tiles, i0 + per);
  auto head = [&](int q) { return (static_cast<int64_t>(sb.cu[b] + (r0 + q) / rep) * H + g * rep + (r0 + q) % rep); };
  for (int i = threadIdx.x; i < kWaQ * D; i += blockDim.x) sq[i] = i / D < cnt ? ldf(qx + head(i / D) * D + i % D) : 0.f;
  for (int i = threadIdx.x; i < kWaQ * DV; i += blockDim.x) so[i] = 0.f;
  float m[kWaMine], l[kWaMine];
  int pos[kWaMine], first[kWaMine];        // position of the pair's token (-1: no pair), blocks that it sees
#pragma unroll
  for (int j = 0; j < kWaMine; ++j) {
    const int q = warp + j * kWaWarps;
    m[j] = -INFINITY;
    l[j] = 0.f;
    pos[j] = q < cnt ? start + (r0 + q) / rep : -1;
    first[j] = blocks ? blocks_seen(pos[j], mask.size, mask.pool) : 0;
  }
  for (int it = i0; it < i1; ++it) {
    const int k0 = (it < n_keep ? it : w0 + it - n_keep) * kWaK;
    const bool means = blocks && it < n_keep;
    __syncthreads();
    for (int k = warp; k < kWaK; k += kWaWarps) {
      const int64_t row = means ? (k0 + k < kept ? pooled_row(pages, mask.pool, slot, k0 + k) : -1)
                                : (k0 + k <= p_hi ? page_row(pages, slot, k0 + k) : -1);
      const T* base = (means ? pooled : static_cast<const T*>(pages.pool)) + (row < 0 ? 0 : row) * pages.width;
      stage_row(base + g * D, row >= 0, D, lane, sk + k * DS);
      stage_row(base + G * D + g * DV, row >= 0, DV, lane, sv + k * DV);
    }
    __syncthreads();
    float s[kWaMine];
#pragma unroll
    for (int j = 0; j < kWaMine; ++j) s[j] = 0.f;
    const float* kv = sk + lane * DS;
    const float* qv = sq + warp * D;
#pragma unroll 4
    for (int i = 0; i < D; ++i) {
      const float kk = kv[i];
#pragma unroll
      for (int j = 0; j < kWaMine; ++j) s[j] = fmaf(qv[j * kWaWarps * D + i], kk, s[j]);
    }
    float a[kWaMine];
#pragma unroll
    for (int j = 0; j < kWaMine; ++j) {
      const int kp = k0 + lane;
      const bool seen = means ? kp < first[j] : kp <= pos[j] && (pos[j] - kp < mask.size || kp < mask.keep_first);
      float sc = s[j] * score.scale;
      if (score.softcap > 0.f) sc = score.softcap * tanhf(sc / score.softcap);
      if (!seen) sc = -INFINITY;
      const float mn = fmaxf(m[j], warp_max(sc));
      const float ref = mn == -INFINITY ? 0.f : mn;   // nothing seen yet: every weight below is 0
      const float p = expf(sc - ref);
      a[j] = expf(m[j] - ref);
      l[j] = l[j] * a[j] + warp_sum(p);
      m[j] = mn;
      sp[(warp + j * kWaWarps) * kWaK + lane] = p;
    }
    __syncwarp();
    for (int c = lane; c < DV; c += 32) {
      float o[kWaMine];
#pragma unroll
      for (int j = 0; j < kWaMine; ++j) o[j] = so[(warp + j * kWaWarps) * DV + c] * a[j];
#pragma unroll 8
      for (int k = 0; k < kWaK; ++k) {
        const float v = sv[k * DV + c];
#pragma unroll
        for (int j = 0; j < kWaMine; ++j) o[j] = fmaf(sp[(warp + j * kWaWarps) * kWaK + k], v, o[j]);
      }
#pragma unroll
      for (int j = 0; j < kWaMine; ++j) so[(warp + j * kWaWarps) * DV + c] = o[j];
    }
  }
  if (i1 <= i0) __syncthreads();           // no tile in this range: the zeroed outputs below must be visible
#pragma unroll
  for (int j = 0; j < kWaMine; ++j) {
    const int q = warp + j * kWaWarps;
    if (q >= cnt) continue;
    const int64_t nh = head(q);
    if (S == 1) {
      float den = l[j], f = 1.f;
      if (score.sink != nullptr) {
        const float sk = score.sink[g * rep + (r0 + q) % rep], mm = fmaxf(m[j], sk);
        f = expf(m[j] - mm);
        den = den * f + expf(sk - mm);
      }
      const float w = f / den;
      for (int c = lane; c < DV; c += 32) stf(out + nh * DV + c, so[q * DV + c] * w);
    } else {
      for (int c = lane; c < DV; c += 32) part_o[(nh * S + split) * DV + c] = so[q * DV + c];
      if (lane == 0) {
        part_ml[(nh * S + split) * 2] = m[j];
        part_ml[(nh * S + split) * 2 + 1] = l[j];
      }
    }
  }
}

template <typename T>
__global__ void window_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, const float* __restrict__ sink,
                                    int H, int D, int S, T* __restrict__ out) {
  const int64_t nh = blockIdx.x;
  float mm = sink != nullptr ? sink[nh % H] : -INFINITY;
  for (int s = 0; s < S; ++s) mm = fmaxf(mm, part_ml[(nh * S + s) * 2]);
  float den = sink != nullptr ? expf(sink[nh % H] - mm) : 0.f;
  for (int s = 0; s < S; ++s) den += part_ml[(nh * S + s) * 2 + 1] * expf(part_ml[(nh * S + s) * 2] - mm);
  for (int c = threadIdx.x; c < D; c += blockDim.x) {
    float v = 0.f;
    for (int s = 0; s < S; ++s) {
      const float ms = part_ml[(nh * S + s) * 2];
      if (ms != -INFINITY) v += part_o[(nh * S + s) * D + c] * expf(ms - mm);
    }
    stf(out + nh * D + c, v / den);
  }
}

template <typename T>
cudaError_t window_attention_t(const SeqBatch& sb, const T* q, const PagedRows& pages, const T* pooled, int H, int G, int D, int DV,
                               WindowMask mask, const ScoreArgs& score, int n_splits, float* part_o, float* part_ml, T* out,
                               cudaStream_t st) {
  static int have = 0;
  const int smem = 4 * (kWaK * ((D | 1) + DV) + kWaQ * (D + DV) + kWaQ * kWaK);
  cudaError_t e = want_smem(window_attn_kernel<T>, smem, have);
  if (e != cudaSuccess) return e;
  const dim3 grid(static_cast<unsigned>(static_cast<int64_t>(sb.n_tok) * (H / G) / kWaQ + sb.n_seq), n_splits, G);
  window_attn_kernel<T><<<grid, kWaWarps * 32, smem, st>>>(sb, q, pages, pooled, H, G, D, DV, mask, score, part_o, part_ml, out);
  if (n_splits > 1) window_merge_kernel<T><<<sb.n_tok * H, 128, 0, st>>>(part_o, part_ml, score.sink, H, DV, n_splits, out);
  return cudaGetLastError();
}

}  // namespace

cudaError_t launch_qk_prepare(bool f32, const SeqBatch& sb, const void* y, int64_t ldy, const float* bias, int H, int G, int D,
                              bool unit_norm, float eps, const RopeTable& rope, const PagedRows& pages, void* q, void* k, void* v,
                              int* status, cudaStream_t st) {
  if (pages.width != 2 * G * D || rope.dims > D) return cudaErrorInvalidValue;
  const PrepArgs a{sb, bias, H, G, D, eps, unit_norm ? 1 : 0, rope, pages, ldy, status};
  const int64_t units = static_cast<int64_t>(sb.n_tok) * (H + G);
  if (f32) {
    qk_prepare_kernel<float><<<static_cast<unsigned>((units + 7) / 8), 256, 0, st>>>(
        a, static_cast<const float*>(y), static_cast<float*>(q), static_cast<float*>(k), static_cast<float*>(v));
    return cudaGetLastError();
  }
  using B = __nv_bfloat16;
  const B* yb = static_cast<const B*>(y);
  B *qb = static_cast<B*>(q), *kb = static_cast<B*>(k), *vb = static_cast<B*>(v);
  const bool vec = D % 16 == 0 && rope.dims % 16 == 0 && D <= 512 && ldy % 8 == 0 &&
                   ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(bias) | reinterpret_cast<uintptr_t>(rope.cos) |
                     reinterpret_cast<uintptr_t>(rope.sin)) & 15) == 0;
#define B200_PREP(L) \
  qk_prepare_vec_kernel<L><<<static_cast<unsigned>((units + 256 / L - 1) / (256 / L)), 256, 0, st>>>(a, yb, qb, kb, vb)
  if (vec && D <= 64) B200_PREP(4);
  else if (vec && D <= 128) B200_PREP(8);
  else if (vec && D <= 256) B200_PREP(16);
  else if (vec) B200_PREP(32);
  else qk_prepare_kernel<B><<<static_cast<unsigned>((units + 7) / 8), 256, 0, st>>>(a, yb, qb, kb, vb);
#undef B200_PREP
  return cudaGetLastError();
}

cudaError_t launch_window_attention(bool f32, const SeqBatch& sb, const void* q, const PagedRows& pages, const void* pooled, int H, int G,
                                    int D, int DV, WindowMask mask, const ScoreArgs& score, int n_splits, float* part_o, float* part_ml,
                                    void* out, cudaStream_t st) {
  if (G < 1 || H % G != 0 || pages.width != G * (D + DV) || mask.size < 1 || mask.keep_first < 0 || n_splits < 1 || mask.pool < 0 ||
      (mask.pool > 0 && (pooled == nullptr || mask.keep_first > 0)) || (n_splits > 1 && (part_o == nullptr || part_ml == nullptr)))
    return cudaErrorInvalidValue;
  using B = __nv_bfloat16;
  return f32 ? window_attention_t<float>(sb, static_cast<const float*>(q), pages, static_cast<const float*>(pooled), H, G, D, DV, mask, score,
                                         n_splits, part_o, part_ml, static_cast<float*>(out), st)
             : window_attention_t<B>(sb, static_cast<const B*>(q), pages, static_cast<const B*>(pooled), H, G, D, DV, mask, score, n_splits,
                                     part_o, part_ml, static_cast<B*>(out), st);
}

}  // namespace b200
