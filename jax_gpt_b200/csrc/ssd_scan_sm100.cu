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
constexpr int kCd = 4;                             // chunks whose c_j are kept
constexpr int kOffXp = kStages * kStageBytes;      // X' high, X' low
constexpr int kOffS = kOffXp + 2 * kXBytes;        // S high, S low
constexpr int kOffBar = kOffS + 2 * kXBytes;
constexpr uint32_t kColG = 0, kColY = 256, kColT = 320, kColYo = 384;   // G: two buffers of 128 columns

struct SsdShared {
  uint64_t full[kStages], empty[kStages], g_full[2], m_ready[2], c_full[kCd], xp_ready, y_full, s_ready;
  uint32_t tmem_base;
  int abort_flag;
  float part[4];
  alignas(16) float e[kL];                         // c_j - log2(dt_j) of the chunk in work: L_ij = 2^(c_i - e_j)
  alignas(16) float c[kCd][kL];                    // c_j in log2 units; the chunk warps run ahead of the state warps
};
constexpr int kSmem = kOffBar + ((sizeof(SsdShared) + 15) & ~15);   // the window starts 1024-byte aligned (checked)
static_assert(kSmem <= 227 * 1024, "shared memory");

struct SsdArgs {
  SeqBatch sb;
  const __nv_bfloat16* dt_raw;
  int64_t ld_dt;
  const float* dt_bias;
  const float* a_log;
  const float* d_skip;
  float* state;
  __nv_bfloat16* y;
  SsdShape s;
  int* status;
};

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

__global__ void __launch_bounds__(kThreads, 1)
ssd_scan_sm100_kernel(const __grid_constant__ CUtensorMap t_xbc, const __grid_constant__ SsdArgs a) {
  extern __shared__ __align__(1024) uint8_t smem[];
  SsdShared* sh = reinterpret_cast<SsdShared*>(smem + kOffBar);
  volatile int* abort_flag = &sh->abort_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int halves = a.s.P / kP;
  const int h = blockIdx.x / halves, p0 = (blockIdx.x % halves) * kP, b = blockIdx.y;
  const int first = a.sb.cu[b], len = a.sb.cu[b + 1] - first;
  const int n_chunks = (len + kL - 1) / kL;
  const int inner = a.s.H * a.s.P;
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
      const int g = h / (a.s.H / a.s.G);
      const int col_b = inner + g * kN, col_c = inner + a.s.G * kN + g * kN, col_x = h * a.s.P + p0;
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
    const float bias = a.dt_bias[h], decay = -expf(a.a_log[h]) * 1.4426950408889634f, dsk = a.d_skip[h];
    auto load_dt = [&](int n) -> float {
      const int t = n * kL + r;
      return t < len ? __bfloat162float(a.dt_raw[static_cast<int64_t>(first + t) * a.ld_dt + h]) : 0.f;
    };
    float raw = load_dt(0);
    bool ok = true;
    // `ok` may differ between warps after a timeout, but every warp runs every iteration with all its barriers
    for (int n = 0; n < n_chunks; ++n) {
      const float dt = n * kL + r < len ? softplus_f(raw + bias) : 0.f;
      float cum = dt * decay;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float t = __shfl_up_sync(0xffffffffu, cum, o);
        if (lane >= o) cum += t;
      }
      if (half == 0 && lane == 31) sh->part[q] = cum;
      if (n + 1 < n_chunks) raw = load_dt(n + 1);
      chunk_sync();   // every warp is done with e of chunk n - 1
      float c_end = 0.f;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float t = sh->part[k];
        if (k < q) cum += t;
        c_end += t;
      }
      if (half == 0) {
        sh->c[n & (kCd - 1)][r] = cum;
        sh->e[r] = cum - log2f(dt);
        mbar_arrive(&sh->c_full[n & (kCd - 1)]);
      }
      chunk_sync();
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
              float f[4] = {__uint_as_float(v[j]) * ex2(cum - e.x), __uint_as_float(v[j + 1]) * ex2(cum - e.y),
                            __uint_as_float(v[j + 2]) * ex2(cum - e.z), __uint_as_float(v[j + 3]) * ex2(cum - e.w)};
#pragma unroll
              for (int k = 0; k < 4; ++k) {
                const int d = r - (j0 + j + k);
                f[k] = d > 0 ? f[k] : (d == 0 ? f[k] + dsk : 0.f);
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
      // ---- X' (its buffer is free once the products of chunk n - 1 are done) ----
      if (ok && n > 0 && !mbar_wait(&sh->y_full, (n - 1) & 1, abort_flag)) {
        if (lane == 0) report_status(a.status, kWaitTmemFullTimeout, 317, h, n);
        ok = false;
      }
      if (ok && !mbar_wait(&sh->full[n & 1], (n >> 1) & 1, abort_flag)) ok = false;
      ok = __all_sync(0xffffffffu, ok);
      if (ok) {
        const uint8_t* tx = smem + (n & 1) * kStageBytes + 2 * kTileBytes;
        const float w = ex2(c_end - cum) * dt;
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
    }
  } else {
    // ---- state warps: S operand, outputs, state update ----
    constexpr int kHalf = kP / 2;
    const int q = warp & 3, half = (warp - 2 - kGroup / 32) >> 2;
    const int r = q * 32 + lane;   // row of the state, and token of the outputs
    const uint32_t lane_off = static_cast<uint32_t>(q * 32) << 16;
    uint8_t* s_hi = smem + kOffS;
    uint8_t* s_lo = s_hi + kXBytes;
    float* gs = a.state + ((static_cast<int64_t>(a.sb.ids[b]) * a.s.H + h) * kN + r) * a.s.P + p0 + half * kHalf;
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
      if (ok && (!mbar_wait(&sh->c_full[n & (kCd - 1)], (n / kCd) & 1, abort_flag) || !mbar_wait(&sh->y_full, n & 1, abort_flag))) {
        if (lane == 0) report_status(a.status, kWaitTmemFullTimeout, 318, h, n);
        ok = false;
      }
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) continue;
      tc_fence_after();
      const float* c = sh->c[n & (kCd - 1)];
      const float ei = ex2(c[r]), ee = ex2(c[kL - 1]);
      const int t = n * kL + r;
      __nv_bfloat16* yo = a.y + static_cast<int64_t>(first + t) * inner + h * a.s.P + p0 + half * kHalf;
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

}  // namespace

bool ssd_scan_sm100_ok(const SsdShape& s) {
  return s.N == kN && s.P >= kP && s.P % kP == 0 && s.G >= 1 && s.H % s.G == 0;
}

cudaError_t launch_ssd_scan_sm100(const SeqBatch& sb, const __nv_bfloat16* xbc, const __nv_bfloat16* dt_raw, int64_t ld_dt,
                                  const float* dt_bias, const float* a_log, const float* d_skip, float* state,
                                  __nv_bfloat16* y, const SsdShape& s, int* status, cudaStream_t st) {
  if (!ssd_scan_sm100_ok(s)) return cudaErrorInvalidValue;
  const uint64_t cols = static_cast<uint64_t>(s.H) * s.P + 2ull * s.G * s.N;
  CUtensorMap m;
  cudaError_t e = encode_tma_2d(&m, xbc, 2, cols, sb.n_tok, cols * 2, 64, kL);
  if (e != cudaSuccess) return e;
  static bool configured = false;
  if (!configured) {
    e = cudaFuncSetAttribute(ssd_scan_sm100_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  const SsdArgs a{sb, dt_raw, ld_dt, dt_bias, a_log, d_skip, state, y, s, status};
  ssd_scan_sm100_kernel<<<dim3(s.H * (s.P / kP), sb.n_seq), kThreads, kSmem, st>>>(m, a);
  return cudaGetLastError();
}

}  // namespace b200
