// Chunked state-space recurrence (Mamba-2, "state-space duality") on tcgen05 tensor cores, bf16 activations with
// fp32 state:
//   S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t      (S is N x P, N = 128)
// One CTA per (64 columns of a head, sequence) walks chunks of 128 tokens. With c_i = the running sum of
// -exp(A_log) dt inside the chunk and L_ij = exp(c_i - c_j) dt_j for j <= i, else 0:
//   G = C B^T,  M = G * L + D I,  Y = M X                              (inside the chunk, skip term included)
//   Yo = C S                                                           (S the state the chunk starts from)
//   T = B^T X'  with X'_j = exp(c_end - c_j) dt_j x_j
//   y_i = Y_i + exp(c_i) Yo_i,   S <- exp(c_end) S + T
// B, C and X enter the products as the bf16 values they are; the fp32 operands (M, S, X') are split into a high and a
// low bf16 part, so the products carry about 16 mantissa bits of them and the sums are fp32. M goes back to TMEM over
// G as the A operand; S and X' are B operands in shared memory (S high | low side by side as one 128-wide operand).
//
// Only S links the chunks, so the work is a pipeline over chunks: warp 0 loads tiles by TMA (two stages), warp 1 issues
// the MMAs, eight "chunk" warps turn G(n + 1) into M and X into X' while eight "state" warps finish chunk n (outputs,
// state update, next S operand); G is double-buffered in TMEM. A tail chunk reads rows of the next sequence (or the
// zero fill): their step sizes count as 0, so they neither decay nor feed the state, and their outputs are not stored.
// Step sizes, decays and exponentials are fp32 (this file is built without fast-math).
//
// The same pipeline runs linear attention with queries, keys and values per head (C = q, B = k, X = v, no skip term):
//  * kDecay: a fixed decay per head, c_i = (i + 1) log(decay), step sizes 1;
//  * kGated: exponential gates with a running maximum (linear_attention.cu). With F_i the running sum of the log forget
//    gates inside the chunk, g_j = i_j - F_j, m0 the maximum the chunk starts with and P_i = max(m0, g_0 .. g_i):
//    m_i = F_i + P_i, L_ij = exp(g_j - P_i), and the state enters row i with exp(m0 - P_i) and the next chunk with
//    exp(m0 - P_end). The chunk warps of a head's first column block also carry the normaliser n: n . q is the row sum of
//    M plus the weighted dot product with n, and n <- exp(m0 - P_end) n + sum_j exp(g_j - P_end) k_j. The outputs are the
//    numerators; their denominators' parts go to `den`.
#include "serve_kernels.cuh"

#include "serve_common.cuh"
#include "tma_host.h"

namespace b200 {

namespace {

constexpr int kL = 128, kN = 128, kP = 64;
constexpr int kTileBytes = kL * kN * 2;            // 32 KB: 128 x 128 bf16 as two 64-column blocks of 16 KB
constexpr int kXBytes = kL * kP * 2;               // 16 KB
constexpr int kStages = 2;
constexpr int kStageBytes = 2 * kTileBytes + kXBytes;   // C | B | X
constexpr int kGroup = 256;                        // threads of the chunk warps, and of the state warps
constexpr int kThreads = 64 + 2 * kGroup;
constexpr int kCd = 3;                             // chunks whose c_j are kept: the chunk warps may be two ahead
constexpr int kOffXp = kStages * kStageBytes;      // X' high, X' low
constexpr int kOffS = kOffXp + 2 * kXBytes;        // S high, S low
constexpr int kOffBar = kOffS + 2 * kXBytes;
constexpr uint32_t kColG = 0, kColY = 256, kColT = 320, kColYo = 384;   // G: two buffers of 128 columns

struct SsdShared {
  uint64_t full[kStages], empty[kStages], g_full[2], m_ready[2], c_full[kCd], xp_ready, y_full, s_ready;
  uint32_t tmem_base;
  int abort_flag;
  float part[4], part2[4], c_end[kCd];             // c_end: log2 of the state's factor over the chunk
  alignas(16) float e[kL];                         // c_j - log2(dt_j) of the chunk in work: L_ij = 2^(c_i - e_j)
  alignas(16) float c[kCd][kL];                    // log2 of the factor with which the state enters row i
  alignas(16) float nv[kN];                        // normaliser at the chunk's start
};
constexpr int kSmem = kOffBar + ((sizeof(SsdShared) + 15) & ~15);   // the window starts 1024-byte aligned (checked)
static_assert(kSmem <= 227 * 1024, "shared memory");

enum ScanMode { kSsd, kDecay, kGated };
constexpr float kLog2e = 1.4426950408889634f;

struct ScanArgs {
  SeqBatch sb;
  int H, P, rep;                   // rep: heads that share a C and B column block
  int col_c, col_b, col_x;         // first columns of C (q), B (k) and X (v) in the input rows
  const __nv_bfloat16* dt_raw;     // kSsd
  int64_t ld_dt;
  const float* dt_bias;
  const float* a_log;
  const float* d_skip;
  LinGates g;                      // kDecay, kGated
  float q_scale;
  float* state;
  __nv_bfloat16* y;
  int* status;
};

__device__ __forceinline__ float warp_prefix_max(float v) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float t = __shfl_up_sync(0xffffffffu, v, o);
    if (lane >= o) v = fmaxf(v, t);
  }
  return v;
}
__device__ __forceinline__ float warp_prefix_sum(float v) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float t = __shfl_up_sync(0xffffffffu, v, o);
    if (lane >= o) v += t;
  }
  return v;
}

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void chunk_sync() { asm volatile("bar.sync 1, %0;" ::"n"(kGroup) : "memory"); }

__device__ __forceinline__ void tmem_ld_x16(uint32_t taddr, uint32_t (&v)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]),
        "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
      : "r"(taddr)
      : "memory");
}

// byte offset of (row r, column c < 64) in a bf16 tile of 128-byte swizzled rows
__device__ __forceinline__ uint32_t swz(int r, int c) { return r * 128 + (((c >> 3) ^ (r & 7)) << 4) + (c & 7) * 2; }

// v[0..7] as a high bf16 part and the bf16 rounding of the remainder
__device__ __forceinline__ void split8(const float* v, uint4& hi, uint4& lo) {
  uint32_t h[4], l[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    h[j] = pack_bf16x2(v[2 * j], v[2 * j + 1]);
    const float2 f = unpack_bf16x2(h[j]);
    l[j] = pack_bf16x2(v[2 * j] - f.x, v[2 * j + 1] - f.y);
  }
  hi = make_uint4(h[0], h[1], h[2], h[3]);
  lo = make_uint4(l[0], l[1], l[2], l[3]);
}

template <int kMode>
__global__ void __launch_bounds__(kThreads, 1)
chunk_scan_kernel(const __grid_constant__ CUtensorMap t_xbc, const __grid_constant__ ScanArgs a) {
  extern __shared__ __align__(1024) uint8_t smem[];
  SsdShared* sh = reinterpret_cast<SsdShared*>(smem + kOffBar);
  volatile int* abort_flag = &sh->abort_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int halves = a.P / kP;
  const int h = blockIdx.x / halves, p0 = (blockIdx.x % halves) * kP, b = blockIdx.y;
  const int first = a.sb.cu[b], len = a.sb.cu[b + 1] - first;
  const int n_chunks = (len + kL - 1) / kL;
  const int inner = a.H * a.P;
  if ((smem_u32(smem) & 1023) != 0) {
    if (threadIdx.x == 0) report_status(a.status, kBadArgument, 315, smem_u32(smem));
    return;
  }

  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) {
      mbar_init(&sh->full[s], 1);
      mbar_init(&sh->empty[s], 1);
      mbar_init(&sh->g_full[s], 1);
      mbar_init(&sh->m_ready[s], kGroup);   // per buffer: the chunk warps may be a chunk ahead of the MMA warp
    }
    for (int s = 0; s < kCd; ++s) mbar_init(&sh->c_full[s], kL);
    mbar_init(&sh->xp_ready, kGroup);
    mbar_init(&sh->y_full, 1);
    mbar_init(&sh->s_ready, kGroup);
    sh->abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(&sh->tmem_base, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sh->tmem_base;

  if (warp == 0) {
    if (lane == 0) {
      const int g = h / a.rep;
      const int col_b = a.col_b + g * kN, col_c = a.col_c + g * kN, col_x = a.col_x + h * a.P + p0;
      int issued = 0;
      bool ok = true;
      for (int n = 0; n < n_chunks; ++n, ++issued) {
        const int st = n & 1;
        if (n >= kStages && !mbar_wait(&sh->empty[st], ((n >> 1) - 1) & 1, abort_flag)) {
          report_status(a.status, kWaitEmptyTimeout, 310, h, n);
          ok = false;
          break;
        }
        uint8_t* base = smem + st * kStageBytes;
        const int row = first + n * kL;
        mbar_arrive_expect_tx(&sh->full[st], kStageBytes);
        tma_load_2d(base, &t_xbc, &sh->full[st], col_c, row);
        tma_load_2d(base + 16384, &t_xbc, &sh->full[st], col_c + 64, row);
        tma_load_2d(base + kTileBytes, &t_xbc, &sh->full[st], col_b, row);
        tma_load_2d(base + kTileBytes + 16384, &t_xbc, &sh->full[st], col_b + 64, row);
        tma_load_2d(base + 2 * kTileBytes, &t_xbc, &sh->full[st], col_x, row);
      }
      if (!ok || *abort_flag) {   // leave no bulk copy in flight (bounded)
        const uint64_t tw = globaltimer_ns();
        for (int s = 0; s < kStages; ++s) {
          const int uses = (issued + 1 - s) / 2;
          if (uses > 0)
            while (!mbar_try_wait(&sh->full[s], (uses - 1) & 1) && globaltimer_ns() - tw < 2000000ull) {
            }
        }
      }
    }
  } else if (warp == 1) {
    constexpr uint32_t i_kk = make_idesc(128, 128, 0, 0, 1);    // G: C (K-major) x B (K-major)
    constexpr uint32_t i_yo = make_idesc(128, 128, 0, 1, 1);    // Yo: C (K-major) x [S high | S low] (MN-major)
    constexpr uint32_t i_y = make_idesc(128, kP, 0, 1, 1);      // Y: M (TMEM) x X (MN-major)
    constexpr uint32_t i_t = make_idesc(128, kP, 1, 1, 1);      // T: B (MN-major) x X' (MN-major)
    const uint32_t a_s = smem_u32(smem + kOffS), a_xp = smem_u32(smem + kOffXp);
    auto tile = [&](int n) { return smem_u32(smem + (n & 1) * kStageBytes); };
    auto issue_g = [&](int n) -> bool {
      if (!mbar_wait(&sh->full[n & 1], (n >> 1) & 1, abort_flag)) {
        if (lane == 0) report_status(a.status, kWaitFullTimeout, 311, h, n);
        return false;
      }
      tc_fence_after();
      if (lane == 0) {
        const uint32_t tc = tile(n), tb = tc + kTileBytes;
#pragma unroll
        for (int k = 0; k < 8; ++k)   // K = state size
          umma_bf16(tmem + kColG + (n & 1) * 128, make_smem_desc(tc + (k >> 2) * 16384 + (k & 3) * 32, 16, 1024),
                    make_smem_desc(tb + (k >> 2) * 16384 + (k & 3) * 32, 16, 1024), i_kk, k > 0 ? 1u : 0u);
        tc_commit(&sh->g_full[n & 1]);
      }
      __syncwarp();
      return true;
    };
    const bool ok = issue_g(0);
    for (int n = 0; ok && n < n_chunks; ++n) {
      // G(n + 1) goes into the buffer of M(n - 1), whose product Y(n - 1) was issued before and runs first
      if (n + 1 < n_chunks && !issue_g(n + 1)) break;
      const uint32_t tc = tile(n), tb = tc + kTileBytes, tx = tb + kTileBytes;
      if (!mbar_wait(&sh->s_ready, n & 1, abort_flag)) {
        if (lane == 0) report_status(a.status, kWaitFullTimeout, 312, h, n);
        break;
      }
      tc_fence_after();
      if (lane == 0) {
#pragma unroll
        for (int k = 0; k < 8; ++k)   // K = state size; the second 64 columns are the low parts
          umma_bf16(tmem + kColYo, make_smem_desc(tc + (k >> 2) * 16384 + (k & 3) * 32, 16, 1024),
                    make_smem_desc(a_s + k * 2048, 16384, 1024), i_yo, k > 0 ? 1u : 0u);
      }
      __syncwarp();
      if (!mbar_wait(&sh->m_ready[n & 1], (n >> 1) & 1, abort_flag)) {
        if (lane == 0) report_status(a.status, kWaitFullTimeout, 313, h, n);
        break;
      }
      tc_fence_after();
      if (lane == 0) {
#pragma unroll
        for (int k = 0; k < 16; ++k)   // K = tokens; step k of M: high words at 16 k, low words at 16 k + 8
          umma_bf16_ts(tmem + kColY, tmem + kColG + (n & 1) * 128 + (k >> 1) * 16 + (k & 1) * 8,
                       make_smem_desc(tx + (k >> 1) * 2048, 16384, 1024), i_y, k > 0 ? 1u : 0u);
      }
      __syncwarp();
      if (!mbar_wait(&sh->xp_ready, n & 1, abort_flag)) {
        if (lane == 0) report_status(a.status, kWaitFullTimeout, 314, h, n);
        break;
      }
      tc_fence_after();
      if (lane == 0) {
#pragma unroll
        for (int k = 0; k < 16; ++k)   // K = tokens, X' high then low
          umma_bf16(tmem + kColT, make_smem_desc(tb + (k & 7) * 2048, 16384, 1024),
                    make_smem_desc(a_xp + (k >> 3) * kXBytes + (k & 7) * 2048, 16384, 1024), i_t, k > 0 ? 1u : 0u);
        tc_commit(&sh->empty[n & 1]);
        tc_commit(&sh->y_full);
      }
      __syncwarp();
    }
  } else if (warp < 2 + kGroup / 32) {
    // ---- chunk warps: step sizes, M, X' ----
    const int q = warp & 3, half = (warp - 2) >> 2;
    const int r = q * 32 + lane;   // token of the chunk
    const uint32_t lane_off = static_cast<uint32_t>(q * 32) << 16;
    uint8_t* xp_hi = smem + kOffXp;
    uint8_t* xp_lo = xp_hi + kXBytes;
    const int64_t row0 = first;
    const bool own = kMode == kGated && p0 == 0;
    float bias = 0.f, decay = 0.f, dsk = 0.f, ibias = 0.f, lq = 0.f, m0 = 0.f;
    const int64_t vec_at = (static_cast<int64_t>(a.sb.ids[b]) * a.H + h) * (kN + 1);
    if constexpr (kMode == kSsd) {
      bias = a.dt_bias[h];
      decay = -expf(a.a_log[h]) * kLog2e;
      dsk = a.d_skip[h];
    } else if constexpr (kMode == kDecay) {
      decay = log2f(a.g.decay[h]);
      lq = log2f(a.q_scale);
    } else {
      ibias = a.g.bias[h];
      bias = a.g.bias[a.H + h];
      lq = log2f(a.q_scale);
      const bool carried = a.sb.start[b] > 0;
      if (carried) m0 = a.g.vec[vec_at + kN] * kLog2e;
      if (half == 0) sh->nv[r] = carried ? a.g.vec[vec_at + r] : 0.f;
    }
    // raw gate inputs of a row: (step size, -) or (input gate, forget gate)
    auto load_raw = [&](int n) -> float2 {
      const int64_t t = n * kL + r;
      if (kMode == kDecay || t >= len) return make_float2(0.f, 0.f);
      if constexpr (kMode == kSsd) return make_float2(__bfloat162float(a.dt_raw[(row0 + t) * a.ld_dt + h]), 0.f);
      const float* p = a.g.raw + (row0 + t) * a.g.ld + h;
      return make_float2(p[0], p[a.H]);
    };
    float2 raw = load_raw(0);
    bool ok = true;
    int cd = 0;                    // n % kCd
    // `ok` may differ between warps after a timeout, but every warp runs every iteration with all its barriers
    for (int n = 0; n < n_chunks; ++n) {
      const bool valid = n * kL + r < len;
      float dt = 1.f, gin = 0.f, cum = 0.f;
      if constexpr (kMode == kSsd) {
        dt = valid ? softplus_f(raw.x + bias) : 0.f;
        cum = dt * decay;
      } else if constexpr (kMode == kGated) {
        gin = valid ? a.g.cap * tanhf((raw.x + ibias) / a.g.cap) * kLog2e : -INFINITY;
        cum = valid ? -softplus_f(-a.g.cap * tanhf((raw.y + bias) / a.g.cap)) * kLog2e : 0.f;
      }
      if constexpr (kMode != kDecay) {
        cum = warp_prefix_sum(cum);
        if (half == 0 && lane == 31) sh->part[q] = cum;
      }
      if (n + 1 < n_chunks) raw = load_raw(n + 1);
      chunk_sync();   // every warp is done with e of chunk n - 1
      float c_end = 0.f;
      if constexpr (kMode == kDecay) {
        const int cnt = min(kL, len - n * kL);
        cum = decay * min(r + 1, cnt);
        c_end = decay * cnt;
      } else {
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float t = sh->part[k];
          if (k < q) cum += t;
          c_end += t;
        }
      }
      float row_c = cum + lq, row_s = row_c, w = 0.f;   // log2 factors of row r of M and of the state; weight of X'
      float e_r = 0.f, f_end = 0.f, p_end = 0.f, p_r = 0.f;
      if constexpr (kMode == kSsd) {
        e_r = cum - log2f(dt);
        w = ex2(c_end - cum) * dt;
      } else if constexpr (kMode == kDecay) {
        e_r = valid ? cum : INFINITY;
        w = valid ? ex2(c_end - cum) : 0.f;
      } else {
        f_end = c_end;
        const float g = gin - cum;
        p_r = warp_prefix_max(g);
        if (half == 0 && lane == 31) sh->part2[q] = p_r;
        chunk_sync();
        p_end = m0;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float t = sh->part2[k];
          if (k < q) p_r = fmaxf(p_r, t);
          p_end = fmaxf(p_end, t);
        }
        p_r = fmaxf(p_r, m0);
        e_r = -g;
        row_c = lq - p_r;
        row_s = row_c + m0;
        c_end = m0 - p_end;
        w = ex2(g - p_end);
      }
      if (half == 0) {
        sh->c[cd][r] = row_s;
        if (r == 0) sh->c_end[cd] = c_end;
        sh->e[r] = e_r;
        mbar_arrive(&sh->c_full[cd]);
      }
      chunk_sync();
      float row_sum = 0.f;
      // ---- M over G, sixteen columns at a time (the two warps of a row take alternate groups) ----
      if (ok && !mbar_wait(&sh->g_full[n & 1], (n >> 1) & 1, abort_flag)) {
        if (lane == 0) report_status(a.status, kWaitTmemFullTimeout, 316, h, n);
        ok = false;
      }
      ok = __all_sync(0xffffffffu, ok);
      if (ok) {
        tc_fence_after();
        const uint32_t tg = tmem + kColG + (n & 1) * 128 + lane_off;
#pragma unroll 1
        for (int gi = half; gi < 8; gi += 2) {
          const int j0 = gi * 16;
          uint32_t v[16], m[16];
          if (j0 <= q * 32 + 31) {   // warp-uniform: part of the group is at or below the diagonal
            tmem_ld_x16(tg + j0, v);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; j += 4) {
              const float4 e = *reinterpret_cast<const float4*>(&sh->e[j0 + j]);
              float f[4] = {__uint_as_float(v[j]) * ex2(row_c - e.x), __uint_as_float(v[j + 1]) * ex2(row_c - e.y),
                            __uint_as_float(v[j + 2]) * ex2(row_c - e.z), __uint_as_float(v[j + 3]) * ex2(row_c - e.w)};
#pragma unroll
              for (int k = 0; k < 4; ++k) {
                const int d = r - (j0 + j + k);
                if constexpr (kMode == kSsd) f[k] = d > 0 ? f[k] : (d == 0 ? f[k] + dsk : 0.f);
                else f[k] = d >= 0 ? f[k] : 0.f;
                if constexpr (kMode == kGated) row_sum += f[k];
              }
#pragma unroll
              for (int k = 0; k < 4; k += 2) {
                const uint32_t hw = pack_bf16x2(f[k], f[k + 1]);
                const float2 u = unpack_bf16x2(hw);
                m[(j + k) / 2] = hw;
                m[8 + (j + k) / 2] = pack_bf16x2(f[k] - u.x, f[k + 1] - u.y);
              }
            }
          } else {
#pragma unroll
            for (int j = 0; j < 16; ++j) m[j] = 0u;
          }
          tmem_st_32x16(tg + j0, m);
        }
        tmem_st_wait();
        tc_fence_before();
      }
      mbar_arrive(&sh->m_ready[n & 1]);
      if (ok && !mbar_wait(&sh->full[n & 1], (n >> 1) & 1, abort_flag)) ok = false;
      ok = __all_sync(0xffffffffu, ok);
      if constexpr (kMode == kGated) {
        if (own) {
          const uint8_t* tq = smem + (n & 1) * kStageBytes;
          const uint8_t* tk = tq + kTileBytes;
          float acc[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[j] = 0.f;
          // this warp's 16 columns of n: two chunks of eight, every sixteenth row per lane pair
          const int cc = 2 * (warp - 2) + (lane & 1), sl = lane >> 1;
          const int rbase = ((sl & 3) << 1) | ((sl >> 2) & 1) | (sl & 8);
          if (ok) {
            // n . q over this half's 64 features
            float dot = 0.f;
#pragma unroll
            for (int c = 0; c < 8; ++c) {
              float x[8];
              Vec16<__nv_bfloat16>::load(reinterpret_cast<const __nv_bfloat16*>(tq + half * 16384 + swz(r, c * 8)), x);
#pragma unroll
              for (int j = 0; j < 8; j += 4) {
                const float4 nv = *reinterpret_cast<const float4*>(&sh->nv[half * 64 + c * 8 + j]);
                dot += (x[j] * nv.x + x[j + 1] * nv.y) + (x[j + 2] * nv.z + x[j + 3] * nv.w);
              }
            }
            if (valid) {
              float* d = a.g.den + ((row0 + n * kL + r) * a.H + h) * 4;
              d[half] = fmaf(ex2(row_s), dot, row_sum);
              if (half == 0) d[2] = ex2(-(cum + p_r));
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              const int row = rbase + 16 * i;
              const float wj = ex2(-sh->e[row] - p_end);
              float x[8];
              Vec16<__nv_bfloat16>::load(reinterpret_cast<const __nv_bfloat16*>(tk + (cc >> 3) * 16384 + swz(row, (cc & 7) * 8)), x);
#pragma unroll
              for (int j = 0; j < 8; ++j) acc[j] = fmaf(wj, x[j], acc[j]);
            }
          }
          // sum over the sixteen row slices; a lane pair ends up with one column
          float s4[4], s2[2];
          const bool h4 = lane & 16, h3 = lane & 8, h2 = lane & 4;
#pragma unroll
          for (int j = 0; j < 4; ++j)
            s4[j] = (h4 ? acc[j + 4] : acc[j]) + __shfl_xor_sync(0xffffffffu, h4 ? acc[j] : acc[j + 4], 16);
#pragma unroll
          for (int j = 0; j < 2; ++j) s2[j] = (h3 ? s4[j + 2] : s4[j]) + __shfl_xor_sync(0xffffffffu, h3 ? s4[j] : s4[j + 2], 8);
          float sum = (h2 ? s2[1] : s2[0]) + __shfl_xor_sync(0xffffffffu, h2 ? s2[0] : s2[1], 4);
          sum += __shfl_xor_sync(0xffffffffu, sum, 2);
          chunk_sync();   // every thread has read n of this chunk
          if ((lane & 2) == 0) {
            float& v = sh->nv[cc * 8 + (h4 ? 4 : 0) + (h3 ? 2 : 0) + (h2 ? 1 : 0)];
            v = fmaf(v, ex2(c_end), sum);
          }
        }
        m0 = f_end + p_end;
      }
      // ---- X' (its buffer is free once the products of chunk n - 1 are done) ----
      if (ok && n > 0 && !mbar_wait(&sh->y_full, (n - 1) & 1, abort_flag)) {
        if (lane == 0) report_status(a.status, kWaitTmemFullTimeout, 317, h, n);
        ok = false;
      }
      ok = __all_sync(0xffffffffu, ok);
      if (ok) {
        const uint8_t* tx = smem + (n & 1) * kStageBytes + 2 * kTileBytes;
#pragma unroll
        for (int j = 0; j < kP / 2; j += 8) {
          const uint32_t o = swz(r, half * (kP / 2) + j);
          const uint4 v = *reinterpret_cast<const uint4*>(tx + o);
          const float2 f0 = unpack_bf16x2(v.x), f1 = unpack_bf16x2(v.y), f2 = unpack_bf16x2(v.z), f3 = unpack_bf16x2(v.w);
          const float f[8] = {f0.x * w, f0.y * w, f1.x * w, f1.y * w, f2.x * w, f2.y * w, f3.x * w, f3.y * w};
          uint4 hi, lo;
          split8(f, hi, lo);
          *reinterpret_cast<uint4*>(xp_hi + o) = hi;
          *reinterpret_cast<uint4*>(xp_lo + o) = lo;
        }
        fence_proxy_async_smem();
      }
      mbar_arrive(&sh->xp_ready);
      if (++cd == kCd) cd = 0;
    }
    if constexpr (kMode == kGated) {
      if (own) {   // other blocks of the head may still read the slot's old values: head_norm_gate moves these there
        chunk_sync();
        float* vn = a.g.vec_new + (static_cast<int64_t>(b) * a.H + h) * (kN + 1);
        if (half == 0) vn[r] = sh->nv[r];
        if (half == 0 && r == 0) vn[kN] = m0 / kLog2e;
      }
    }
  } else {
    // ---- state warps: S operand, outputs, state update ----
    constexpr int kHalf = kP / 2;
    const int q = warp & 3, half = (warp - 2 - kGroup / 32) >> 2;
    const int r = q * 32 + lane;   // row of the state, and token of the outputs
    const uint32_t lane_off = static_cast<uint32_t>(q * 32) << 16;
    uint8_t* s_hi = smem + kOffS;
    uint8_t* s_lo = s_hi + kXBytes;
    float* gs = a.state + ((static_cast<int64_t>(a.sb.ids[b]) * a.H + h) * kN + r) * a.P + p0 + half * kHalf;
    float S[kHalf];
    if (a.sb.start[b] > 0) {
#pragma unroll
      for (int j = 0; j < kHalf; j += 4) {
        const float4 f = *reinterpret_cast<const float4*>(gs + j);
        S[j] = f.x; S[j + 1] = f.y; S[j + 2] = f.z; S[j + 3] = f.w;
      }
    } else {
#pragma unroll
      for (int j = 0; j < kHalf; ++j) S[j] = 0.f;
    }
    bool ok = true;
    int cd = 0;
    uint32_t cd_phase = 0;
    for (int n = 0; n < n_chunks; ++n) {
#pragma unroll
      for (int j = 0; j < kHalf; j += 8) {
        uint4 hi, lo;
        split8(S + j, hi, lo);
        const uint32_t o = swz(r, half * kHalf + j);
        *reinterpret_cast<uint4*>(s_hi + o) = hi;
        *reinterpret_cast<uint4*>(s_lo + o) = lo;
      }
      fence_proxy_async_smem();
      mbar_arrive(&sh->s_ready);
      if (ok && (!mbar_wait(&sh->c_full[cd], cd_phase, abort_flag) || !mbar_wait(&sh->y_full, n & 1, abort_flag))) {
        if (lane == 0) report_status(a.status, kWaitTmemFullTimeout, 318, h, n);
        ok = false;
      }
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) continue;
      tc_fence_after();
      const float ei = ex2(sh->c[cd][r]), ee = ex2(sh->c_end[cd]);
      if (++cd == kCd) {
        cd = 0;
        cd_phase ^= 1;
      }
      const int t = n * kL + r;
      __nv_bfloat16* yo = a.y + static_cast<int64_t>(first + t) * inner + h * a.P + p0 + half * kHalf;
      const uint32_t tc = tmem + half * kHalf + lane_off;
#pragma unroll
      for (int g = 0; g < kHalf; g += 16) {
        uint32_t v[16], hi[16], lo[16];
        tmem_ld_x16(tc + kColT + g, v);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 16; ++j) S[g + j] = fmaf(S[g + j], ee, __uint_as_float(v[j]));
        tmem_ld_x16(tc + kColY + g, v);
        tmem_ld_x16(tc + kColYo + g, hi);
        tmem_ld_x16(tc + kColYo + kP + g, lo);
        tmem_ld_wait();
        if (t < len) {
          uint32_t o[8];
#pragma unroll
          for (int j = 0; j < 8; ++j)
            o[j] = pack_bf16x2(
                fmaf(ei, __uint_as_float(hi[2 * j]) + __uint_as_float(lo[2 * j]), __uint_as_float(v[2 * j])),
                fmaf(ei, __uint_as_float(hi[2 * j + 1]) + __uint_as_float(lo[2 * j + 1]), __uint_as_float(v[2 * j + 1])));
          *reinterpret_cast<uint4*>(yo + g) = make_uint4(o[0], o[1], o[2], o[3]);
          *reinterpret_cast<uint4*>(yo + g + 8) = make_uint4(o[4], o[5], o[6], o[7]);
        }
      }
      tc_fence_before();
    }
    if (ok) {
#pragma unroll
      for (int j = 0; j < kHalf; j += 4) *reinterpret_cast<float4*>(gs + j) = make_float4(S[j], S[j + 1], S[j + 2], S[j + 3]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

template <int kMode>
cudaError_t launch_chunk_scan(const __nv_bfloat16* x, int64_t ld, uint64_t cols, const ScanArgs& a, cudaStream_t st) {
  CUtensorMap m;
  cudaError_t e = encode_tma_2d(&m, x, 2, cols, a.sb.n_tok, ld * 2, 64, kL);
  if (e != cudaSuccess) return e;
  static bool configured = false;
  if (!configured) {
    e = cudaFuncSetAttribute(chunk_scan_kernel<kMode>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  chunk_scan_kernel<kMode><<<dim3(a.H * (a.P / kP), a.sb.n_seq), kThreads, kSmem, st>>>(m, a);
  return cudaGetLastError();
}

}  // namespace

bool ssd_scan_sm100_ok(const SsdShape& s) {
  return s.N == kN && s.P >= kP && s.P % kP == 0 && s.G >= 1 && s.H % s.G == 0;
}

cudaError_t launch_ssd_scan_sm100(const SeqBatch& sb, const __nv_bfloat16* xbc, const __nv_bfloat16* dt_raw, int64_t ld_dt,
                                  const float* dt_bias, const float* a_log, const float* d_skip, float* state,
                                  __nv_bfloat16* y, const SsdShape& s, int* status, cudaStream_t st) {
  if (!ssd_scan_sm100_ok(s)) return cudaErrorInvalidValue;
  const int inner = s.H * s.P, cols = inner + 2 * s.G * s.N;
  ScanArgs a{};
  a.sb = sb;
  a.H = s.H;
  a.P = s.P;
  a.rep = s.H / s.G;
  a.col_x = 0;
  a.col_b = inner;
  a.col_c = inner + s.G * s.N;
  a.dt_raw = dt_raw;
  a.ld_dt = ld_dt;
  a.dt_bias = dt_bias;
  a.a_log = a_log;
  a.d_skip = d_skip;
  a.q_scale = 1.f;
  a.state = state;
  a.y = y;
  a.status = status;
  return launch_chunk_scan<kSsd>(xbc, cols, cols, a, st);
}

bool linear_scan_sm100_ok(const LinShape& s) { return s.N == kN && s.P >= kP && s.P % kP == 0 && s.q_scale > 0.f && s.silu == 0; }

cudaError_t launch_linear_scan_sm100(const SeqBatch& sb, const __nv_bfloat16* qkv, int64_t ld, const LinGates& g, float* state,
                                     __nv_bfloat16* y, const LinShape& s, int* status, cudaStream_t st) {
  if (!linear_scan_sm100_ok(s) || ld % 8 != 0 || (reinterpret_cast<uintptr_t>(qkv) & 15) != 0) return cudaErrorInvalidValue;
  ScanArgs a{};
  a.sb = sb;
  a.H = s.H;
  a.P = s.P;
  a.rep = 1;
  a.col_c = 0;
  a.col_b = s.H * s.N;
  a.col_x = 2 * s.H * s.N;
  a.g = g;
  a.q_scale = s.q_scale;
  a.state = state;
  a.y = y;
  a.status = status;
  const uint64_t cols = static_cast<uint64_t>(s.H) * (2 * s.N + s.P);
  return g.raw != nullptr ? launch_chunk_scan<kGated>(qkv, ld, cols, a, st) : launch_chunk_scan<kDecay>(qkv, ld, cols, a, st);
}

}  // namespace b200
