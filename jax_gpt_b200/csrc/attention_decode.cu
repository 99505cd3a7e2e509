// Single-token (decode) attention over a dense KV cache laid out as (B, Hkv, max_len, D), split over the keys.
//
// Decode attention is a stream over the cache: every key and value row is read once for the G = H / Hkv query
// heads that share it, and there are at most eight query rows per kv head, far too few for a tensor-core tile. So
// this is a bandwidth kernel: a CTA takes one (key range, kv head, sequence); D/8 lanes share a key row with one
// 16-byte load each, dot it with the G queries held in registers, reduce across those lanes with shuffles and run
// an online softmax per lane group; groups, warps and finally key ranges are merged by their (max, sum) pairs.
// The number of valid keys may come from a device counter, so a CUDA-graph decode loop needs no host value.
//
// Replaces the dense masked attention over the whole cache buffer of the reference's cached paths
// (jax_gpt/models/qwen35/gqa.py:88-119, jax_gpt/models/gpt2/model.py:159-176).
#include "attention_sm100.cuh"

#include "common.cuh"
#include "softcap.cuh"

namespace b200 {

namespace {

constexpr int kDecWarps = 4;

struct DecArgs {
  const __nv_bfloat16* q;   // [B, H*D], row stride ldq
  int64_t ldq;
  const __nv_bfloat16* k;   // cache (B, Hkv, max_len, D): strides in elements
  const __nv_bfloat16* v;
  int64_t kv_stride_b, kv_stride_h, kv_stride_t;
  const int* pos_ptr;       // device: number of valid keys = pos_ptr[0] + len_add (nullptr: len)
  int len, len_add;
  int H, Hkv;
  float scale_log2;
  float* part_o;            // [B, H, n_splits, D] un-normalised partial outputs
  float* part_ml;           // [B, H, n_splits, 2] (running max in log2 units, sum)
  // paged cache (table != nullptr): k / v point at the K and V halves of a page pool [n_pages, page_size, width];
  // key t of sequence seq_ids[b] sits in row table[seq, t / page_size] * page_size + t % page_size, kv_stride_t is the
  // pool's row width, the number of valid keys is lens[seq] + len_add
  const int* table;
  const int* seq_ids;
  const int* lens;
  int page_size, max_pages;
  int window, keep_first;   // window > 0: of the valid keys only the last `window` and the first `keep_first` are seen
  int64_t v_stride_h;       // between the kv heads of V
  // pool > 0 (paged, keep_first 0): the mean rows of the blocks of `pool` tokens that lie wholly before the window are seen too; they sit
  // in pages of ceil(page_size / pool) rows, in the page of a block's last token
  const __nv_bfloat16* pooled;
  int pool;
  SoftCap cap;              // kCap instances
};

// D: query and key width, DV: value width (D or 2 D).
template <int D, int DV, int G, bool kCap, bool kPool>
__global__ void __launch_bounds__(kDecWarps * 32)
attn_decode_split_kernel(const DecArgs a) {
  constexpr int LPK = D / 8;          // lanes that share one key row
  constexpr int KPW = 32 / LPK;       // keys per warp step
  constexpr int KPS = KPW * kDecWarps;
  constexpr int EV = DV / LPK, NV = EV / 8;   // value features of a lane, in 16-byte pieces LPK * 8 features apart
  __shared__ float sm_o[kDecWarps][G][DV];
  __shared__ float sm_m[kDecWarps][G], sm_l[kDecWarps][G];
  const int split = blockIdx.x, hkv = blockIdx.y, b = blockIdx.z;
  const int n_splits = gridDim.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int sub = lane % LPK, grp = lane / LPK;
  const int seq = a.table != nullptr ? a.seq_ids[b] : b;
  const int len = a.table != nullptr ? a.lens[seq] + a.len_add : (a.pos_ptr != nullptr ? a.pos_ptr[0] + a.len_add : a.len);
  const int* pages = a.table != nullptr ? a.table + static_cast<int64_t>(seq) * a.max_pages : nullptr;
  // The seen keys are numbered through: the kept first ones, then the window (which may start among them).
  const int n_keep = kPool ? max(0, len - a.window) / a.pool : (a.window > 0 ? min(a.keep_first, len) : 0);
  const int w0 = a.window > 0 ? max(kPool ? 0 : n_keep, len - a.window) : 0;
  const int n_seen = n_keep + len - w0;
  // cache row of seen key t: its position for a dense cache, page * page_size + offset for a paged one
  const int block_rows = kPool ? (a.page_size + a.pool - 1) / a.pool : 0;
  auto key_row = [&](int t) -> int64_t {
    if (t >= n_keep) {
      t += w0 - n_keep;
    } else if (kPool) {
      const int pi = (t * a.pool + a.pool - 1) / a.page_size;
      return static_cast<int64_t>(pages[pi]) * block_rows + t - pi * a.page_size / a.pool;
    }
    if (pages == nullptr) return t;
    return static_cast<int64_t>(pages[t / a.page_size]) * a.page_size + t % a.page_size;
  };
  const int per = ((n_seen + n_splits - 1) / n_splits + KPS - 1) / KPS * KPS;
  const int k0 = split * per, k1 = min(n_seen, k0 + per);

  float qf[G][8];
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const uint4 u = *reinterpret_cast<const uint4*>(a.q + static_cast<int64_t>(b) * a.ldq + (hkv * G + g) * D + sub * 8);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = unpack_bf16x2(w[e]);
      qf[g][2 * e] = kCap ? f.x : f.x * a.scale_log2;
      qf[g][2 * e + 1] = kCap ? f.y : f.y * a.scale_log2;
    }
  }
  float m[G], l[G], o[G][EV];
#pragma unroll
  for (int g = 0; g < G; ++g) {
    m[g] = -INFINITY;
    l[g] = 0.f;
#pragma unroll
    for (int e = 0; e < EV; ++e) o[g][e] = 0.f;
  }
  const __nv_bfloat16* kb = a.k + b * a.kv_stride_b + hkv * a.kv_stride_h + sub * 8;
  const __nv_bfloat16* vb = a.v + b * a.kv_stride_b + hkv * a.v_stride_h + sub * 8;
  const __nv_bfloat16* kp = kPool ? a.pooled + hkv * a.kv_stride_h + sub * 8 : nullptr;   // the same in the rows of means
  const __nv_bfloat16* vp = kPool ? a.pooled + (a.v - a.k) + hkv * a.v_stride_h + sub * 8 : nullptr;
  // Two keys per lane group in flight. The trip count is uniform over the warp (the shuffles below need every
  // lane); a lane group whose key is past the range loads nothing and skips the update.
  for (int base = k0 + warp * KPW; base < k1; base += 2 * KPS) {
    const int ka = base + grp, kc = ka + KPS;
    const bool has_a = ka < k1, has_c = kc < k1;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    const int64_t ra = has_a ? key_row(ka) * a.kv_stride_t : 0, rc = has_c ? key_row(kc) * a.kv_stride_t : 0;
    const bool pa = kPool && ka < n_keep, pc = kPool && kc < n_keep;
    const __nv_bfloat16 *va = pa ? vp : vb, *vc = pc ? vp : vb;
    const uint4 kua = has_a ? *reinterpret_cast<const uint4*>((pa ? kp : kb) + ra) : zero;
    const uint4 kuc = has_c ? *reinterpret_cast<const uint4*>((pc ? kp : kb) + rc) : zero;
    uint4 vua[NV], vuc[NV];
#pragma unroll
    for (int p = 0; p < NV; ++p) {
      vua[p] = has_a ? *reinterpret_cast<const uint4*>(va + ra + p * D) : zero;
      vuc[p] = has_c ? *reinterpret_cast<const uint4*>(vc + rc + p * D) : zero;
    }
#pragma unroll
    for (int which = 0; which < 2; ++which) {
      const uint4 ku = which == 0 ? kua : kuc;
      const bool valid = which == 0 ? has_a : has_c;
      const uint32_t kw[4] = {ku.x, ku.y, ku.z, ku.w};
      float kf[8], vf[EV];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = unpack_bf16x2(kw[e]);
        kf[2 * e] = f.x;
        kf[2 * e + 1] = f.y;
      }
#pragma unroll
      for (int p = 0; p < NV; ++p) {
        const uint4 vu = which == 0 ? vua[p] : vuc[p];
        const uint32_t vw[4] = {vu.x, vu.y, vu.z, vu.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 f = unpack_bf16x2(vw[e]);
          vf[8 * p + 2 * e] = f.x;
          vf[8 * p + 2 * e + 1] = f.y;
        }
      }
#pragma unroll
      for (int g = 0; g < G; ++g) {
        float s = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) s = fmaf(qf[g][e], kf[e], s);
#pragma unroll
        for (int off = LPK / 2; off > 0; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
        if (kCap) s = soft_cap(s, a.cap);
        if (valid) {
          const float mn = fmaxf(m[g], s);
          const float alpha = exp2f(m[g] - mn), p = exp2f(s - mn);
          l[g] = fmaf(l[g], alpha, p);
#pragma unroll
          for (int e = 0; e < EV; ++e) o[g][e] = fmaf(o[g][e], alpha, p * vf[e]);
          m[g] = mn;
        }
      }
    }
  }
  // merge the lane groups of a warp (same columns, different keys)
#pragma unroll
  for (int off = LPK; off < 32; off <<= 1) {
#pragma unroll
    for (int g = 0; g < G; ++g) {
      const float mo = __shfl_xor_sync(0xffffffffu, m[g], off);
      const float lo = __shfl_xor_sync(0xffffffffu, l[g], off);
      const float mn = fmaxf(m[g], mo);
      const float wa = (m[g] == -INFINITY) ? 0.f : exp2f(m[g] - mn);
      const float wb = (mo == -INFINITY) ? 0.f : exp2f(mo - mn);
      l[g] = l[g] * wa + lo * wb;
#pragma unroll
      for (int e = 0; e < EV; ++e) {
        const float oo = __shfl_xor_sync(0xffffffffu, o[g][e], off);
        o[g][e] = o[g][e] * wa + oo * wb;
      }
      m[g] = mn;
    }
  }
  if (grp == 0) {
#pragma unroll
    for (int g = 0; g < G; ++g) {
#pragma unroll
      for (int e = 0; e < EV; ++e) sm_o[warp][g][(e / 8) * D + sub * 8 + e % 8] = o[g][e];
      if (sub == 0) {
        sm_m[warp][g] = m[g];
        sm_l[warp][g] = l[g];
      }
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < G * DV; i += kDecWarps * 32) {
    const int g = i / DV, c = i % DV;
    float mn = -INFINITY;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) mn = fmaxf(mn, sm_m[w][g]);
    float acc = 0.f, ls = 0.f;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) {
      const float wt = (sm_m[w][g] == -INFINITY) ? 0.f : exp2f(sm_m[w][g] - mn);
      acc = fmaf(sm_o[w][g][c], wt, acc);
      ls = fmaf(sm_l[w][g], wt, ls);
    }
    const int64_t row = (static_cast<int64_t>(b) * a.H + hkv * G + g) * n_splits + split;
    a.part_o[row * DV + c] = acc;
    if (c == 0) {
      a.part_ml[row * 2] = mn;
      a.part_ml[row * 2 + 1] = ls;
    }
  }
}

// out[b, h, :] = sum_s part_o[s] 2^(m_s - M) / (sum_s l_s 2^(m_s - M) + the sink's weight); one CTA per (head, sequence). The
// ranges' weights go through shared memory; kGroups groups of D threads each sum every kGroups-th range.
constexpr int kMaxSplits = 256;

template <int D>
__global__ void __launch_bounds__(512)
attn_decode_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, int n_splits,
                         __nv_bfloat16* __restrict__ out, int64_t ldo, int H, const float* __restrict__ sink) {
  constexpr int kGroups = 512 / D;
  __shared__ float wt[kMaxSplits], acc_s[kGroups][D], red[1];
  const int h = blockIdx.x, b = blockIdx.y, c = threadIdx.x % D, grp = threadIdx.x / D;
  const int64_t row0 = (static_cast<int64_t>(b) * H + h) * n_splits;
  if (threadIdx.x < 32) {
    const float sk = sink != nullptr ? sink[h] * 1.4426950408889634f : -INFINITY;
    float mn = sk, ls = 0.f;
    for (int s = threadIdx.x; s < n_splits; s += 32) mn = fmaxf(mn, part_ml[(row0 + s) * 2]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, o));
    for (int s = threadIdx.x; s < n_splits; s += 32) {
      const float ms = part_ml[(row0 + s) * 2];
      const float w = (ms == -INFINITY) ? 0.f : exp2f(ms - mn);
      wt[s] = w;
      ls = fmaf(part_ml[(row0 + s) * 2 + 1], w, ls);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ls += __shfl_xor_sync(0xffffffffu, ls, o);
    if (threadIdx.x == 0) red[0] = ls + (sink != nullptr ? exp2f(sk - mn) : 0.f);
  }
  __syncthreads();
  float acc = 0.f;
#pragma unroll 8
  for (int s = grp; s < n_splits; s += kGroups) acc = fmaf(part_o[(row0 + s) * D + c], wt[s], acc);
  acc_s[grp][c] = acc;
  __syncthreads();
  if (grp == 0) {
#pragma unroll
    for (int g = 1; g < kGroups; ++g) acc += acc_s[g][c];
    const float ls = red[0];
    out[static_cast<int64_t>(b) * ldo + h * D + c] = __float2bfloat16(ls > 0.f ? acc / ls : 0.f);
  }
}

template <int D, int DV, int G>
cudaError_t decode_launch(const DecArgs& a, int B, int n_splits, __nv_bfloat16* out, int64_t ldo,
                          cudaStream_t stream, const float* sink) {
  const bool cap = a.cap.out > 0.f;
  if (n_splits > kMaxSplits || (a.pool > 0 && cap)) return cudaErrorInvalidValue;
  dim3 grid(n_splits, a.Hkv, B);
  if (a.pool > 0) attn_decode_split_kernel<D, DV, G, false, true><<<grid, kDecWarps * 32, 0, stream>>>(a);
  else if (cap) attn_decode_split_kernel<D, DV, G, true, false><<<grid, kDecWarps * 32, 0, stream>>>(a);
  else attn_decode_split_kernel<D, DV, G, false, false><<<grid, kDecWarps * 32, 0, stream>>>(a);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return e;
  attn_decode_merge_kernel<DV><<<dim3(a.H, B), 512, 0, stream>>>(a.part_o, a.part_ml, n_splits, out, ldo, a.H, sink);
  return cudaGetLastError();
}

template <int D, int DV = D>
cudaError_t decode_dispatch_g(const DecArgs& a, int B, int n_splits, __nv_bfloat16* out, int64_t ldo,
                              cudaStream_t stream, const float* sink = nullptr) {
  switch (a.H / a.Hkv) {
    case 1: return decode_launch<D, DV, 1>(a, B, n_splits, out, ldo, stream, sink);
    case 2: return decode_launch<D, DV, 2>(a, B, n_splits, out, ldo, stream, sink);
    case 4: return decode_launch<D, DV, 4>(a, B, n_splits, out, ldo, stream, sink);
    case 8: return decode_launch<D, DV, 8>(a, B, n_splits, out, ldo, stream, sink);
    default: return cudaErrorInvalidValue;
  }
}

}  // namespace

cudaError_t launch_attn_decode(const __nv_bfloat16* q, int64_t ldq, const __nv_bfloat16* k, const __nv_bfloat16* v,
                               int64_t kv_stride_b, int64_t kv_stride_h, int64_t kv_stride_t, const int* pos_ptr,
                               int len, int len_add, int B, int H, int Hkv, int D, float scale, int n_splits,
                               float* part_o, float* part_ml, __nv_bfloat16* out, int64_t ldo, cudaStream_t stream) {
  if (H % Hkv != 0 || n_splits < 1 || kv_stride_t % 8 != 0 || kv_stride_h % 8 != 0 || kv_stride_b % 8 != 0 ||
      ldq % 8 != 0)
    return cudaErrorInvalidValue;
  DecArgs a{q, ldq, k, v, kv_stride_b, kv_stride_h, kv_stride_t, pos_ptr, len, len_add, H, Hkv,
            scale * 1.4426950408889634f, part_o, part_ml, nullptr, nullptr, nullptr, 0, 0, 0, 0, kv_stride_h, nullptr, 0, SoftCap{0.f, 0.f}};
  switch (D) {
    case 64: return decode_dispatch_g<64>(a, B, n_splits, out, ldo, stream);
    case 128: return decode_dispatch_g<128>(a, B, n_splits, out, ldo, stream);
    case 256: return decode_dispatch_g<256>(a, B, n_splits, out, ldo, stream);
    default: return cudaErrorInvalidValue;
  }
}

cudaError_t launch_attn_decode_paged(const __nv_bfloat16* q, int64_t ldq, const __nv_bfloat16* pool, int width,
                                     const int* block_table, const int* seq_ids, const int* seq_lens, int len_add,
                                     int page_size, int max_pages, int B, int H, int Hkv, int D, float scale, int n_splits,
                                     float* part_o, float* part_ml, __nv_bfloat16* out, int64_t ldo, cudaStream_t stream,
                                     int window, int keep_first, int DV, const DecodeScores& sc) {
  if (DV == 0) DV = D;
  if (sc.pool > 0 && (sc.pooled == nullptr || window < 1 || keep_first > 0)) return cudaErrorInvalidValue;
  if (H % Hkv != 0 || n_splits < 1 || width != Hkv * (D + DV) || width % 8 != 0 || ldq % 8 != 0 || page_size < 1 || keep_first < 0)
    return cudaErrorInvalidValue;
  // a pool row holds K of every kv head, then V of every kv head
  DecArgs a{q, ldq, pool, pool + Hkv * D, 0, D, width, nullptr, 0, len_add, H, Hkv,
            scale * 1.4426950408889634f, part_o, part_ml, block_table, seq_ids, seq_lens, page_size, max_pages,
            window, keep_first};
  a.v_stride_h = DV;
  a.pooled = sc.pooled;
  a.pool = sc.pool;
  if (sc.softcap > 0.f) a.cap = SoftCap{2.f * 1.4426950408889634f * scale / sc.softcap, sc.softcap * 1.4426950408889634f};
  if (DV == 2 * D && D == 64) return decode_dispatch_g<64, 128>(a, B, n_splits, out, ldo, stream, sc.sink);
  if (DV == 2 * D && D == 128) return decode_dispatch_g<128, 256>(a, B, n_splits, out, ldo, stream, sc.sink);
  if (DV != D) return cudaErrorInvalidValue;
  switch (D) {
    case 64: return decode_dispatch_g<64>(a, B, n_splits, out, ldo, stream, sc.sink);
    case 128: return decode_dispatch_g<128>(a, B, n_splits, out, ldo, stream, sc.sink);
    case 256: return decode_dispatch_g<256>(a, B, n_splits, out, ldo, stream, sc.sink);
    default: return cudaErrorInvalidValue;
  }
}

}  // namespace b200
