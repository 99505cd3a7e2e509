// Linear attention with a decay per key channel on packed batches, chunked (Yang et al., "Gated Linear Attention Transformers with
// Hardware-Efficient Training"): S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = q_scale S_t^T q_t. With F the running sum of
// log alpha in a chunk of 64 tokens and S the state before it,
//   o_i   = (q_i exp(F_i))^T S + sum_(j <= i) A_ij v_j,      A_ij = sum_n q_in k_jn exp(F_in - F_jn)
// and the state advances in four steps of 16 tokens, with keys scaled to the end of theirs: S <- diag(exp(T)) S + sum_j (k_j exp(T - F_j)) v_j^T.
// Every exponent that is formed is at most 0, but for the 16 x 16 blocks on the diagonal of A: those are taken relative to the block's
// middle token where its decays allow that, and pair by pair where they are too strong.
//
// Two launches. Nothing in the first depends on the state: a block per chunk and head makes the decays, the scaled queries and keys and
// A, and leaves them as the shared-memory image (rows padded by 16 bytes) that the second one copies in. The second walks the chunks of
// a sequence with the state of a head and 32 or 64 value columns in registers: half of its warps advance the state, the others make
// the outputs from the state before the chunk. Everything that the state and A are made of enters its product as a high and a low bf16
// part; towards the outputs the scaled queries and A are bf16 operands, like the probabilities of the attention kernels, and the state
// again has two parts. mma.sync: the operands of a step are 64 rows high and the state has to come back to registers every step.
//
// This file is built without fast-math and names its fast intrinsics.
#include "serve_common.cuh"
#include "serve_kernels.cuh"

namespace b200 {

namespace {

using Bf = __nv_bfloat16;
constexpr int kC = 64, kSub = 16, kLdA = kC + 8, kPrepThreads = 320, kScanThreads = 512;

struct Image {   // one (chunk, head); offsets in bytes
  int N, ld;     // key width, row stride of the scaled queries and keys
  __host__ __device__ explicit Image(int n) : N(n), ld(n + 8) {}
  __host__ __device__ int rows() const { return kC * ld * 2; }                     // one of queries, keys' high and low part
  __host__ __device__ int a() const { return 3 * rows(); }
  __host__ __device__ int tiles() const { return a() + kC * kLdA * 2; }            // what the scan copies
  __host__ __device__ int bytes() const { return tiles() + kC / kSub * N * 4; }    // and the decay of every 16 tokens, fp32
};

struct Chunk {
  int b, t0, cnt;   // sequence, first token in it, tokens
};
__device__ __forceinline__ Chunk chunk_at(const SeqBatch& sb, int tile) {
  for (int b = 0; b < sb.n_seq; ++b) {
    const int len = sb.cu[b + 1] - sb.cu[b], n = (len + kC - 1) / kC;
    if (tile < n) return {b, tile * kC, min(kC, len - tile * kC)};
    tile -= n;
  }
  return {-1, 0, 0};
}

__device__ __forceinline__ void mma_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  mma_bf16_16816(d, a[0], a[1], a[2], a[3], b0, b1);
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void cp16(void* dst, const void* src, bool live) {   // 16 bytes, zeros where not live
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// barrier of the scan's warps, which reach it from two places
__device__ __forceinline__ void scan_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(kScanThreads) : "memory"); }

// x = hi + lo with both in bf16
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(x - h.x, y - h.y);
}
// log2 sigmoid(z), to fp32 rounding of the logarithm also where the sigmoid is close to 1
__device__ __forceinline__ float log2_sigmoid(float z) {
  const float e = ex2_approx(-kLog2e * fabsf(z));
  const float l = e < 0.03f ? kLog2e * e * (1.f - e * (0.5f - e * (1.f / 3 - e * 0.25f))) : lg2_approx(1.f + e);
  return fmaf(kLog2e, fminf(z, 0.f), -l);
}

// ---- decays, scaled operands, A ------------------------------------------------------------------------------------------
// Sums of log alpha are kept in units of log 2 and run within 16 tokens, so that neighbours' differences stay exact however far the
// chunk has decayed; [kC][N + 8] with rows turned by 8 words every 16 tokens. T(m) below is the sum of all of block m.
__host__ __device__ __forceinline__ int low_ld(int R) { return (R + 15) / 16 * 16 + 8; }
__host__ __device__ __forceinline__ int prep_smem(int N, int R) {
  return (kC * (N + 8) + kC / 16 * 8) * 4 + 4 * kC * (N + 8) * 2 + kC * low_ld(R) * 2;
}

// (hi + lo) times a factor, split again
__device__ __forceinline__ void rescale2(uint32_t& hi, uint32_t& lo, const float2& w) {
  const float2 h = unpack_bf16x2(hi), l = unpack_bf16x2(lo);
  split2((h.x + l.x) * w.x, (h.y + l.y) * w.y, hi, lo);
}

template <int kN>   // key width, 0: any
__global__ void __launch_bounds__(kPrepThreads, 2)
gla_prep_kernel(const SeqBatch sb, const Bf* __restrict__ qkv, int64_t ld, const LinGates gt, const LinShape s, unsigned char* __restrict__ images) {
  extern __shared__ __align__(16) unsigned char smem[];
  const Chunk ch = chunk_at(sb, blockIdx.x);
  if (ch.b < 0) return;
  const int N = kN > 0 ? kN : s.N, h = blockIdx.y, R = gt.R, ldl = low_ld(R), ldn = N + 8;
  const Image im(N);
  unsigned char* img = images + (static_cast<int64_t>(blockIdx.x) * s.H + h) * im.bytes();
  float* sF = reinterpret_cast<float*>(smem);
  // queries scaled from the start of their 16 tokens on, keys to its end; high and low parts
  Bf* sQ = reinterpret_cast<Bf*>(sF + kC * ldn + kC / 16 * 8);   // [kC][ldn], low parts behind
  Bf* sK = sQ + 2 * kC * ldn;                                    // the same
  Bf* sL = sK + 2 * kC * ldn;                                    // [kC][ldl] low-rank rows
  auto row_of = [&](int tok) { return tok * ldn + (tok >> 4) * 8; };
  const int64_t row0 = sb.cu[ch.b] + ch.t0;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3, chunks = N / 8;
  const int cpad = ldl - 8;
  for (int i = tid; i < kC * cpad; i += kPrepThreads) {
    const int k = i / cpad, r = i % cpad;
    sL[k * ldl + r] = k < ch.cnt && r < R ? static_cast<const Bf*>(gt.low)[(row0 + k) * gt.ld_low + r] : __float2bfloat16(0.f);
  }
  for (int i = tid; i < kC * chunks; i += kPrepThreads) {
    const int k = i / chunks, c = i % chunks * 8;
    const Bf* row = qkv + (row0 + k) * ld + h * N + c;
    cp16(sQ + k * ldn + c, k < ch.cnt ? row : qkv, k < ch.cnt);
    cp16(sK + k * ldn + c, k < ch.cnt ? row + s.H * N : qkv, k < ch.cnt);
  }
  cp_commit();
  __syncthreads();
  // ---- running sums of log alpha: a warp per 16 channels (rows of the product w2 low^T) and all tokens; column g of tile m is token
  // 16 (g / 2) + 2 m + g % 2, which gives a lane 16 consecutive tokens of its two channels ----
  if (warp * 16 < N) {
    float z[8][4];
#pragma unroll
    for (int m = 0; m < 8; ++m)
#pragma unroll
      for (int e = 0; e < 4; ++e) z[m][e] = gt.bias2[h * N + warp * 16 + g + 8 * (e / 2)];
    const Bf* w = static_cast<const Bf*>(gt.w2) + (static_cast<int64_t>(h) * N + warp * 16 + g) * R;
    auto pair = [&](const Bf* p, int r) {
      const unsigned short* u = reinterpret_cast<const unsigned short*>(p);
      return (r < R ? static_cast<uint32_t>(u[r]) : 0u) | (r + 1 < R ? static_cast<uint32_t>(u[r + 1]) << 16 : 0u);
    };
    for (int k = 0; k < cpad; k += 16) {
      const int r = k + 2 * t;
      const uint32_t a0 = pair(w, r), a1 = pair(w + 8 * R, r), a2 = pair(w, r + 8), a3 = pair(w + 8 * R, r + 8);
      const Bf* l = sL + ((g >> 1) * 16 + (g & 1)) * ldl + r;
#pragma unroll
      for (int m = 0; m < 8; ++m)
        mma_bf16_16816(z[m], a0, a1, a2, a3, *reinterpret_cast<const uint32_t*>(l + 2 * m * ldl), *reinterpret_cast<const uint32_t*>(l + 2 * m * ldl + 8));
    }
    const int live = ch.cnt - 16 * t;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float F = 0.f;
#pragma unroll
      for (int m = 0; m < 8; ++m)
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          if (2 * m + p < live) F = fmaf(log2_sigmoid(z[m][2 * e + p]), gt.inv_tau, F);
          z[m][2 * e + p] = F;
        }
      float* f = sF + row_of(16 * t) + warp * 16 + g + 8 * e;
#pragma unroll
      for (int m = 0; m < 8; ++m)
#pragma unroll
        for (int p = 0; p < 2; ++p) f[(2 * m + p) * ldn] = z[m][2 * e + p];
    }
  }
  cp_wait_all();
  __syncthreads();
  // ---- scaled queries and keys ----
  auto total = [&](int m, int c) { return *reinterpret_cast<const float2*>(sF + row_of(m * kSub + kSub - 1) + c); };   // T(m)
  if (tid < 2 * N) {   // eight channels, one token of every 16
    const int c = tid % chunks * 8, k = tid / chunks;
    float before[8];   // decay from the chunk's start to the block's, with the queries' scale
#pragma unroll
    for (int j = 0; j < 8; ++j) before[j] = 0.f;
#pragma unroll
    for (int m = 0; m < kC / kSub; ++m) {
      const int at = (m * kSub + k) * ldn + c;
      const uint4 q4 = *reinterpret_cast<const uint4*>(sQ + at), k4 = *reinterpret_cast<const uint4*>(sK + at);
      const uint32_t qw[4] = {q4.x, q4.y, q4.z, q4.w}, kw[4] = {k4.x, k4.y, k4.z, k4.w};
      const float* f = sF + row_of(m * kSub) + k * ldn + c;
      uint32_t qh[4], ql[4], kh[4], kl[4], qi[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 F = *reinterpret_cast<const float2*>(f + 2 * j), T = total(m, c + 2 * j);
        float2 x = unpack_bf16x2(qw[j]), z = unpack_bf16x2(kw[j]);
        x = make_float2(x.x * ex2_approx(F.x), x.y * ex2_approx(F.y));
        z = make_float2(z.x * ex2_approx(T.x - F.x), z.y * ex2_approx(T.y - F.y));
        split2(x.x, x.y, qh[j], ql[j]);
        split2(z.x, z.y, kh[j], kl[j]);
        qi[j] = pack_bf16x2(x.x * s.q_scale * ex2_approx(before[2 * j]), x.y * s.q_scale * ex2_approx(before[2 * j + 1]));
        before[2 * j] += T.x;
        before[2 * j + 1] += T.y;
      }
      *reinterpret_cast<uint4*>(sQ + at) = make_uint4(qh[0], qh[1], qh[2], qh[3]);
      *reinterpret_cast<uint4*>(sQ + kC * ldn + at) = make_uint4(ql[0], ql[1], ql[2], ql[3]);
      *reinterpret_cast<uint4*>(sK + at) = make_uint4(kh[0], kh[1], kh[2], kh[3]);
      *reinterpret_cast<uint4*>(sK + kC * ldn + at) = make_uint4(kl[0], kl[1], kl[2], kl[3]);
      unsigned char* d = img + at * 2;
      *reinterpret_cast<uint4*>(d) = make_uint4(qi[0], qi[1], qi[2], qi[3]);
      *reinterpret_cast<uint4*>(d + im.rows()) = make_uint4(kh[0], kh[1], kh[2], kh[3]);
      *reinterpret_cast<uint4*>(d + 2 * im.rows()) = make_uint4(kl[0], kl[1], kl[2], kl[3]);
    }
  }
  for (int i = tid; i < kC / kSub * N; i += kPrepThreads) reinterpret_cast<float*>(img + im.tiles())[i] = exp2f(sF[row_of(i / N * kSub + kSub - 1) + i % N]);
  __syncthreads();
  // ---- A: a warp per 16 x 16 block, six below the diagonal and four on it ----
  int I, J;
  if (warp < 6) {
    I = warp < 1 ? 1 : warp < 3 ? 2 : 3;
    J = warp - (I == 1 ? 0 : I == 2 ? 1 : 3);
  } else {
    I = J = warp - 6;
  }
  const bool diag = I == J;
  Bf* A = reinterpret_cast<Bf*>(img + im.a()) + I * kSub * kLdA + J * kSub;
  const float *f = sF + row_of(I * kSub), *mid = f + (kSub / 2 - 1) * ldn;
  if (diag) {
    float spread = 0.f;
    for (int c = lane; c < N; c += 32) spread = fmaxf(spread, -f[(kSub - 1) * ldn + c]);
    if (warp_max(spread) > 60.f) {   // too strong for factors that stay in range: pair by pair
      const Bf* x = qkv + (row0 + I * kSub) * ld + h * N;
      const int rows = min(kSub, ch.cnt - I * kSub);
      for (int i = 0; i < kSub; ++i)
        for (int j = 0; j < kSub; ++j) {
          float v = 0.f;
          if (j <= i && i < rows)
            for (int c = lane; c < N; c += 32) v = fmaf(ldf(x + i * ld + c) * ldf(x + j * ld + s.H * N + c), ex2_approx(f[i * ldn + c] - f[j * ldn + c]), v);
          v = warp_sum(v) * s.q_scale;
          if (lane == 0) A[i * kLdA + j] = __float2bfloat16(v);
        }
      return;
    }
  }
  float acc[2][4] = {};
  const int r16 = lane & 15, c8 = (lane >> 4) * 8, q0 = (I * kSub + r16) * ldn + c8, k0 = (J * kSub + (lane & 7) + (lane >> 4) * 8) * ldn + ((lane >> 3) & 1) * 8;
#pragma unroll 2
  for (int kb = 0; kb < N; kb += 16) {
    uint32_t xh[4], xl[4], yh[4], yl[4];   // queries; keys of the two column tiles
    ldsm4(xh, sQ + q0 + kb);
    ldsm4(xl, sQ + kC * ldn + q0 + kb);
    ldsm4(yh, sK + k0 + kb);
    ldsm4(yl, sK + kC * ldn + k0 + kb);
    if (I - J != 1) {
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        const int c = kb + 2 * t + 8 * p;
        float2 w = make_float2(0.f, 0.f);
        if (diag) {           // from the start and the end of the 16 tokens to their middle
          const float2 M = *reinterpret_cast<const float2*>(mid + c), T = total(I, c);
          w = make_float2(ex2_approx(M.x - T.x), ex2_approx(M.y - T.y));
          rescale2(yh[p], yl[p], w);
          rescale2(yh[2 + p], yl[2 + p], w);
          w = make_float2(ex2_approx(-M.x), ex2_approx(-M.y));
        } else {              // across the blocks between J and I
          for (int m = J + 1; m < I; ++m) {
            const float2 T = total(m, c);
            w.x += T.x;
            w.y += T.y;
          }
          w = make_float2(ex2_approx(w.x), ex2_approx(w.y));
        }
        rescale2(xh[2 * p], xl[2 * p], w);
        rescale2(xh[2 * p + 1], xl[2 * p + 1], w);
      }
    }
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      mma_16816(acc[m], xh, yh[2 * m], yh[2 * m + 1]);
      mma_16816(acc[m], xh, yl[2 * m], yl[2 * m + 1]);
      mma_16816(acc[m], xl, yh[2 * m], yh[2 * m + 1]);
    }
  }
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int i = g + 8 * r, j = m * 8 + 2 * t;
      const float v0 = !diag || j <= i ? acc[m][2 * r] * s.q_scale : 0.f, v1 = !diag || j + 1 <= i ? acc[m][2 * r + 1] * s.q_scale : 0.f;
      *reinterpret_cast<uint32_t*>(A + i * kLdA + j) = pack_bf16x2(v0, v1);
    }
}

// ---- scan over the chunks --------------------------------------------------------------------------------------------------
__host__ __device__ __forceinline__ int stage_bytes(int N, int ps) { return Image(N).tiles() + kC * (ps + 8) * 2; }
__host__ __device__ __forceinline__ int scan_smem(int N, int ps) { return 2 * stage_bytes(N, ps) + 2 * 2 * N * (ps + 8) * 2; }

// kN: key width, 0: any; kPs: value columns of a block. Warps 0-7 own 16 keys each, warps 8-15 an output tile of 16 x kPs / 2.
template <int kN, int kPs>
__global__ void __launch_bounds__(kScanThreads)
gla_scan_kernel(const SeqBatch sb, const Bf* __restrict__ qkv, int64_t ld, const unsigned char* __restrict__ images, float* __restrict__ state,
                Bf* __restrict__ y, const LinShape s) {
  extern __shared__ __align__(16) unsigned char smem[];
  constexpr int kLdP = kPs + 8, kTiles = kPs / 8, kHalf = kTiles / 2;
  const int N = kN > 0 ? kN : s.N, P = s.P, h = blockIdx.x, p0 = blockIdx.y * kPs, b = blockIdx.z;
  const Image im(N);
  const int ldn = im.ld, stage = stage_bytes(N, kPs);
  Bf* sS = reinterpret_cast<Bf*>(smem + 2 * stage);        // [2 buffers][high, low][N][kLdP]
  const int first = sb.cu[b], len = sb.cu[b + 1] - first, chunks = (len + kC - 1) / kC;
  int tile0 = 0;
  for (int i = 0; i < b; ++i) tile0 += (sb.cu[i + 1] - sb.cu[i] + kC - 1) / kC;
  const int tid = threadIdx.x, warp = (tid >> 5) & 7, lane = tid & 31, g = lane >> 2, t = lane & 3;
  auto image = [&](int c) { return images + (static_cast<int64_t>(tile0 + c) * s.H + h) * im.bytes(); };
  auto load = [&](int c) {
    unsigned char* d = smem + (c & 1) * stage;
    const unsigned char* src = image(c);
    for (int i = tid * 16; i < im.tiles(); i += kScanThreads * 16) cp16(d + i, src + i, true);
    Bf* sv = reinterpret_cast<Bf*>(d + im.tiles());
    const Bf* v = qkv + 2 * s.H * N + h * P + p0;
    for (int i = tid; i < kC * kTiles; i += kScanThreads) {
      const int r = i / kTiles, cc = i % kTiles * 8;
      const bool live = c * kC + r < len && p0 + cc < P;
      cp16(sv + r * kLdP + cc, live ? v + static_cast<int64_t>(first + c * kC + r) * ld + cc : qkv, live);
    }
    cp_commit();
  };
  load(0);
  const int r16 = lane & 15, c8 = (lane >> 4) * 8;
  if (tid < kScanThreads / 2) {
    // ---- state: keys 16 warp + g, + 8; columns 8 m + 2 t, + 1 ----
    const bool owner = warp * 16 < N;
    float* st = state + (static_cast<int64_t>(sb.ids[b]) * s.H + h) * N * P;
    const bool fresh = sb.start[b] == 0;
    float S[kTiles][4];
    auto each_state = [&](auto&& f) {
#pragma unroll
      for (int m = 0; m < kTiles; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int key = warp * 16 + g + 8 * (e / 2), p = p0 + m * 8 + 2 * t + e % 2;
          f(S[m][e], key, p, owner && p < P);
        }
    };
    each_state([&](float& v, int key, int p, bool live) { v = live && !fresh ? st[static_cast<int64_t>(key) * P + p] : 0.f; });
    auto publish = [&](int buf) {
      if (!owner) return;
      Bf *hi = sS + buf * 2 * N * kLdP, *lo = hi + N * kLdP;
#pragma unroll
      for (int m = 0; m < kTiles; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t a, c;
          split2(S[m][2 * r], S[m][2 * r + 1], a, c);
          const int at = (warp * 16 + g + 8 * r) * kLdP + m * 8 + 2 * t;
          *reinterpret_cast<uint32_t*>(hi + at) = a;
          *reinterpret_cast<uint32_t*>(lo + at) = c;
        }
    };
    publish(0);
    const int tok = (lane & 7) + (lane >> 4) * 8, key = warp * 16 + ((lane >> 3) & 1) * 8;
    for (int c = 0; c < chunks; ++c) {
      float T[kC / kSub][2];
      if (owner) {
        const float* e = reinterpret_cast<const float*>(image(c) + im.tiles()) + warp * 16 + g;
#pragma unroll
        for (int m = 0; m < kC / kSub; ++m) {
          T[m][0] = e[m * N];
          T[m][1] = e[m * N + 8];
        }
      }
      cp_wait_all();
      scan_barrier();                                      // this chunk's operands and state are visible, the other buffers are free
      if (c + 1 < chunks) load(c + 1);
      if (!owner) continue;
      const unsigned char* d = smem + (c & 1) * stage;
      const Bf *kh = reinterpret_cast<const Bf*>(d + im.rows()), *kl = kh + kC * ldn, *sv = reinterpret_cast<const Bf*>(d + im.tiles());
#pragma unroll
      for (int k = 0; k < kC; k += kSub) {
        uint32_t xh[4], xl[4];
#pragma unroll
        for (int m = 0; m < kTiles; ++m)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[m][e] *= T[k / kSub][e / 2];
        ldsm4_t(xh, kh + (k + tok) * ldn + key);
        ldsm4_t(xl, kl + (k + tok) * ldn + key);
#pragma unroll
        for (int m = 0; m < kTiles; m += 2) {
          uint32_t z[4];
          ldsm4_t(z, sv + (k + r16) * kLdP + m * 8 + c8);
          mma_16816(S[m], xh, z[0], z[1]);
          mma_16816(S[m + 1], xh, z[2], z[3]);
          mma_16816(S[m], xl, z[0], z[1]);
          mma_16816(S[m + 1], xl, z[2], z[3]);
        }
      }
      publish((c + 1) & 1);
    }
    each_state([&](float& v, int key, int p, bool live) { if (live) st[static_cast<int64_t>(key) * P + p] = v; });
  } else {
    // ---- outputs: rows 16 mt .., columns nh .. ----
    const int mt = warp >> 1, nh = (warp & 1) * (kPs / 2);
    for (int c = 0; c < chunks; ++c) {
      cp_wait_all();
      scan_barrier();
      if (c + 1 < chunks) load(c + 1);
      const unsigned char* d = smem + (c & 1) * stage;
      const Bf *qh = reinterpret_cast<const Bf*>(d), *A = reinterpret_cast<const Bf*>(d + im.a()), *sv = reinterpret_cast<const Bf*>(d + im.tiles());
      const Bf *sh = sS + (c & 1) * 2 * N * kLdP, *sl = sh + N * kLdP;
      const int cnt = min(kC, len - c * kC);
      if (mt * 16 >= cnt) continue;
      float o[kHalf][4] = {}, o1[kHalf][4] = {};           // separate sums: short chains of dependent products
#pragma unroll
      for (int k = 0; k < kC / 16; ++k) {
        if (k > mt) break;
        uint32_t x[4];
        ldsm4(x, A + (mt * 16 + r16) * kLdA + k * 16 + c8);
#pragma unroll
        for (int m = 0; m < kHalf; m += 2) {
          uint32_t z[4];
          ldsm4_t(z, sv + (k * 16 + r16) * kLdP + nh + m * 8 + c8);
          mma_16816(o[m], x, z[0], z[1]);
          mma_16816(o[m + 1], x, z[2], z[3]);
        }
      }
#pragma unroll
      for (int k = 0; k < N; k += 16) {
        uint32_t x[4];
        ldsm4(x, qh + (mt * 16 + r16) * ldn + k + c8);
#pragma unroll
        for (int m = 0; m < kHalf; m += 2) {
          uint32_t zh[4], zl[4];
          ldsm4_t(zh, sh + (k + r16) * kLdP + nh + m * 8 + c8);
          ldsm4_t(zl, sl + (k + r16) * kLdP + nh + m * 8 + c8);
          mma_16816(o[m], x, zh[0], zh[1]);
          mma_16816(o[m + 1], x, zh[2], zh[3]);
          mma_16816(o1[m], x, zl[0], zl[1]);
          mma_16816(o1[m + 1], x, zl[2], zl[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < kHalf; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int row = mt * 16 + g + 8 * r, p = p0 + nh + m * 8 + 2 * t;
          if (row < cnt && p < P)
            *reinterpret_cast<uint32_t*>(y + (static_cast<int64_t>(first + c * kC + row) * s.H + h) * P + p) =
                pack_bf16x2(o[m][2 * r] + o1[m][2 * r], o[m][2 * r + 1] + o1[m][2 * r + 1]);
        }
    }
  }
}

template <int kN, int kPs>
cudaError_t gla_scan_go(const SeqBatch& sb, const Bf* qkv, int64_t ld, const unsigned char* img, float* state, Bf* y, const LinShape& s, cudaStream_t st) {
  static int have = 0;
  const int smem = scan_smem(s.N, kPs);
  const cudaError_t e = want_smem(gla_scan_kernel<kN, kPs>, smem, have);
  if (e != cudaSuccess) return e;
  gla_scan_kernel<kN, kPs><<<dim3(s.H, (s.P + kPs - 1) / kPs, sb.n_seq), kScanThreads, smem, st>>>(sb, qkv, ld, img, state, y, s);
  return cudaGetLastError();
}

}  // namespace

bool gla_chunked_ok(const LinShape& s, int64_t ld, int R) {
  return s.N % 16 == 0 && s.N <= 128 && s.P % 8 == 0 && ld % 8 == 0 && R <= 64 && s.silu == 0;
}

int64_t gla_chunked_scratch(const SeqBatch& sb, const LinShape& s) {
  return static_cast<int64_t>(sb.n_tok / kC + sb.n_seq) * s.H * Image(s.N).bytes();
}

cudaError_t launch_gla_chunked(const SeqBatch& sb, const Bf* qkv, int64_t ld, const LinGates& g, float* state, Bf* y, const LinShape& s,
                               void* scratch, cudaStream_t st) {
  if (!gla_chunked_ok(s, ld, g.R) || ((reinterpret_cast<uintptr_t>(qkv) | reinterpret_cast<uintptr_t>(scratch) | reinterpret_cast<uintptr_t>(y)) & 15) != 0)
    return cudaErrorInvalidValue;
  const int ps = prep_smem(s.N, g.R);
  unsigned char* img = static_cast<unsigned char*>(scratch);
  cudaError_t e = cudaSuccess;
#define B200_PREP(N)                                                                                            \
  {                                                                                                             \
    static int have = 0;                                                                                        \
    e = want_smem(gla_prep_kernel<N>, ps, have);                                                                \
    if (e != cudaSuccess) return e;                                                                             \
    gla_prep_kernel<N><<<dim3(sb.n_tok / kC + sb.n_seq, s.H), kPrepThreads, ps, st>>>(sb, qkv, ld, g, s, img);  \
  }
  if (s.N == 128) B200_PREP(128)
  else if (s.N == 64) B200_PREP(64)
  else B200_PREP(0)
#undef B200_PREP
  // wide blocks once they fill the SMs, narrow ones for more of them before
  const bool wide = static_cast<int64_t>(s.H) * ((s.P + 63) / 64) * sb.n_seq >= 148;
#define B200_SCAN(N) return wide ? gla_scan_go<N, 64>(sb, qkv, ld, img, state, y, s, st) : gla_scan_go<N, 32>(sb, qkv, ld, img, state, y, s, st)
  if (s.N == 128) B200_SCAN(128);
  if (s.N == 64) B200_SCAN(64);
  B200_SCAN(0);
#undef B200_SCAN
}

}  // namespace b200
