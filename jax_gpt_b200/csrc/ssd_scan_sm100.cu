// Chunked state-space recurrence (Mamba-2, "state-space duality") on tcgen05 tensor cores, bf16 activations with
// fp32 state:
//   S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t      (S is N x P, N = 128)
// One CTA per (head, sequence) walks chunks of 128 tokens with S in the registers of 256 threads (fp32). With
// c_i = the running sum of -exp(A_log) dt inside the chunk and L_ij = exp(c_i - c_j) dt_j for j <= i, else 0:
//   1. G = C B^T,  Yo = C S          (S the state the chunk starts from)
//   2. Y = (G * L) X,  T = B^T X'    (X'_j = exp(c_end - c_j) dt_j x_j)
//   3. y_i = Y_i + exp(c_i) Yo_i + D x_i,   S <- exp(c_end) S + T
// B, C and X enter the products as the bf16 values they are; the fp32 operands (G * L, S, X') are split into a
// high and a low bf16 part and multiplied twice, so the products carry about 16 mantissa bits of them and the sums
// are fp32. G * L goes back to TMEM as the A operand; S and X' are B operands in shared memory. Chunk tiles arrive by
// TMA (double-buffered at P = 64). A tail chunk reads rows of the next sequence (or the zero fill): their step sizes
// count as 0, so they neither decay nor feed the state, and their outputs are not stored.
// Step sizes, decays and exponentials are fp32 (this file is built without fast-math).
#include "serve_kernels.cuh"

#include "serve_common.cuh"
#include "tma_host.h"

namespace b200 {

namespace {

constexpr int kL = 128, kN = 128;
constexpr int kTileBytes = kL * kN * 2;   // 32 KB: 128 x 128 bf16 as two 64-column blocks of 16 KB
constexpr int kThreads = 320;             // TMA warp, MMA warp, eight compute warps
constexpr int kCompute = 256;

template <int P>
struct SsdCfg {
  static constexpr int kStages = P == 64 ? 2 : 1;
  static constexpr int kXBytes = kL * P * 2;
  static constexpr int kStageBytes = 2 * kTileBytes + kXBytes;   // C | B | X
  static constexpr int kOffXp = kStages * kStageBytes;           // X' high, X' low
  static constexpr int kOffS = kOffXp + 2 * kXBytes;             // S high, S low (128 x P each)
  static constexpr int kOffCd = kOffS + 2 * kXBytes;             // float2 [128]: (c_j in log2 units, dt_j)
  static constexpr int kOffBar = kOffCd + kL * 8;
  static constexpr int kSmem = 1024 + kOffBar + 192;
};

struct SsdBars {
  uint64_t full[2], empty[2], g_full, m_ready, y_full, s_ready;
  uint32_t tmem_base;
  int abort_flag;
  float part[4];
};

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
__device__ __forceinline__ void compute_sync() { asm volatile("bar.sync 1, %0;" ::"n"(kCompute) : "memory"); }

// byte offset of (row r, column c) in a bf16 tile of 64-column blocks (16 KB each) with 128-byte swizzled rows
__device__ __forceinline__ uint32_t swz(int r, int c) {
  return (c >> 6) * 16384 + r * 128 + ((((c & 63) >> 3) ^ (r & 7)) << 4) + (c & 7) * 2;
}

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

template <int P>
__global__ void __launch_bounds__(kThreads, 1)
ssd_scan_sm100_kernel(const __grid_constant__ CUtensorMap t_xbc, const __grid_constant__ SsdArgs a) {
  using C = SsdCfg<P>;
  constexpr int kHalf = P / 2;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  SsdBars* bars = reinterpret_cast<SsdBars*>(smem + C::kOffBar);
  volatile int* abort_flag = &bars->abort_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, b = blockIdx.y;
  const int first = a.sb.cu[b], len = a.sb.cu[b + 1] - first;
  const int n_chunks = (len + kL - 1) / kL;
  const int inner = a.s.H * P;

  if (threadIdx.x == 0) {
    for (int s = 0; s < 2; ++s) {
      mbar_init(&bars->full[s], 1);
      mbar_init(&bars->empty[s], 1);
    }
    mbar_init(&bars->g_full, 1);
    mbar_init(&bars->m_ready, kCompute);
    mbar_init(&bars->y_full, 1);
    mbar_init(&bars->s_ready, kCompute);
    bars->abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(&bars->tmem_base, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_base;
  constexpr uint32_t kColG = 0, kColY = 128, kColYo = 256, kColT = 384;   // G is overwritten by (G * L) high | low

  if (warp == 0) {
    if (lane == 0) {
      const int g = h / (a.s.H / a.s.G);
      const int col_b = inner + g * kN, col_c = inner + a.s.G * kN + g * kN;
      int issued = 0;
      bool ok = true;
      for (int n = 0; n < n_chunks; ++n, ++issued) {
        const int st = n % C::kStages;
        if (n >= C::kStages && !mbar_wait(&bars->empty[st], ((n / C::kStages) - 1) & 1, abort_flag)) {
          report_status(a.status, kWaitEmptyTimeout, 310, h, n);
          ok = false;
          break;
        }
        uint8_t* base = smem + st * C::kStageBytes;
        const int row = first + n * kL;
        mbar_arrive_expect_tx(&bars->full[st], C::kStageBytes);
        tma_load_2d(base, &t_xbc, &bars->full[st], col_c, row);
        tma_load_2d(base + 16384, &t_xbc, &bars->full[st], col_c + 64, row);
        tma_load_2d(base + kTileBytes, &t_xbc, &bars->full[st], col_b, row);
        tma_load_2d(base + kTileBytes + 16384, &t_xbc, &bars->full[st], col_b + 64, row);
#pragma unroll
        for (int k = 0; k < P / 64; ++k)
          tma_load_2d(base + 2 * kTileBytes + k * 16384, &t_xbc, &bars->full[st], h * P + k * 64, row);
      }
      if (!ok || *abort_flag) {   // leave no bulk copy in flight (bounded)
        const uint64_t tw = globaltimer_ns();
        for (int s = 0; s < C::kStages; ++s) {
          const int uses = (issued + C::kStages - 1 - s) / C::kStages;
          if (uses > 0)
            while (!mbar_try_wait(&bars->full[s], (uses - 1) & 1) && globaltimer_ns() - tw < 2000000ull) {
            }
        }
      }
    }
  } else if (warp == 1) {
    constexpr uint32_t i_g = make_idesc(128, 128, 0, 0, 1);   // C (K-major) x B (K-major)
    constexpr uint32_t i_kn = make_idesc(128, P, 0, 1, 1);    // A K-major or in TMEM, B MN-major
    constexpr uint32_t i_nn = make_idesc(128, P, 1, 1, 1);    // both MN-major
    const uint32_t a_s = smem_u32(smem + C::kOffS), a_xp = smem_u32(smem + C::kOffXp);
    for (int n = 0; n < n_chunks; ++n) {
      const int st = n % C::kStages;
      const uint32_t tc = smem_u32(smem + st * C::kStageBytes), tb = tc + kTileBytes, tx = tb + kTileBytes;
      if (!mbar_wait(&bars->s_ready, n & 1, abort_flag) || !mbar_wait(&bars->full[st], (n / C::kStages) & 1, abort_flag)) {
        if (lane == 0) report_status(a.status, kWaitFullTimeout, 311, h, n);
        break;
      }
      tc_fence_after();
      if (lane == 0) {
#pragma unroll
        for (int k = 0; k < 8; ++k)   // K = state size
          umma_bf16(tmem + kColG, make_smem_desc(tc + (k >> 2) * 16384 + (k & 3) * 32, 16, 1024),
                    make_smem_desc(tb + (k >> 2) * 16384 + (k & 3) * 32, 16, 1024), i_g, k > 0 ? 1u : 0u);
#pragma unroll
        for (int k = 0; k < 16; ++k)   // state high, then low
          umma_bf16(tmem + kColYo, make_smem_desc(tc + ((k & 7) >> 2) * 16384 + (k & 3) * 32, 16, 1024),
                    make_smem_desc(a_s + (k >> 3) * C::kXBytes + (k & 7) * 2048, 16384, 1024), i_kn, k > 0 ? 1u : 0u);
        tc_commit(&bars->g_full);
      }
      __syncwarp();
      if (!mbar_wait(&bars->m_ready, n & 1, abort_flag)) {
        if (lane == 0) report_status(a.status, kWaitFullTimeout, 312, h, n);
        break;
      }
      tc_fence_after();
      if (lane == 0) {
#pragma unroll
        for (int k = 0; k < 16; ++k)   // K = tokens
          umma_bf16_ts(tmem + kColY, tmem + kColG + (k >> 3) * 64 + (k & 7) * 8,
                       make_smem_desc(tx + (k & 7) * 2048, 16384, 1024), i_kn, k > 0 ? 1u : 0u);
#pragma unroll
        for (int k = 0; k < 16; ++k)
          umma_bf16(tmem + kColT, make_smem_desc(tb + (k & 7) * 2048, 16384, 1024),
                    make_smem_desc(a_xp + (k >> 3) * C::kXBytes + (k & 7) * 2048, 16384, 1024), i_nn, k > 0 ? 1u : 0u);
        tc_commit(&bars->empty[st]);
        tc_commit(&bars->y_full);
      }
      __syncwarp();
    }
  } else {
    const int q = warp & 3, half = (warp - 2) >> 2;
    const int r = q * 32 + lane;   // row of every TMEM tile owned by this thread: a token of the chunk, or a state row
    const uint32_t lane_off = static_cast<uint32_t>(q * 32) << 16;
    float2* cd = reinterpret_cast<float2*>(smem + C::kOffCd);
    uint8_t* s_hi = smem + C::kOffS;
    uint8_t* s_lo = s_hi + C::kXBytes;
    uint8_t* xp_hi = smem + C::kOffXp;
    uint8_t* xp_lo = xp_hi + C::kXBytes;
    float* gs = a.state + ((static_cast<int64_t>(a.sb.ids[b]) * a.s.H + h) * kN + r) * P + half * kHalf;
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
    const float bias = a.dt_bias[h], decay = -expf(a.a_log[h]) * 1.4426950408889634f, dsk = a.d_skip[h];
    auto load_dt = [&](int n) -> float {
      const int t = n * kL + r;
      return (half == 0 && t < len) ? __bfloat162float(a.dt_raw[static_cast<int64_t>(first + t) * a.ld_dt + h]) : 0.f;
    };
    float raw = load_dt(0);
    bool ok = true;
    // ok may differ between warps after a timeout, but every compute warp runs every iteration with all its barriers
    for (int n = 0; n < n_chunks; ++n) {
      const int st = n % C::kStages;
      // ---- publish the state the chunk starts from ----
#pragma unroll
      for (int j = 0; j < kHalf; j += 8) {
        uint4 hi, lo;
        split8(S + j, hi, lo);
        const uint32_t o = swz(r, half * kHalf + j);
        *reinterpret_cast<uint4*>(s_hi + o) = hi;
        *reinterpret_cast<uint4*>(s_lo + o) = lo;
      }
      fence_proxy_async_smem();
      mbar_arrive(&bars->s_ready);
      // ---- step sizes and running log-decays of the chunk ----
      float cum = 0.f, dt = 0.f;
      if (half == 0) {
        dt = n * kL + r < len ? softplus_f(raw + bias) : 0.f;
        cum = dt * decay;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float t = __shfl_up_sync(0xffffffffu, cum, o);
          if (lane >= o) cum += t;
        }
        if (lane == 31) bars->part[q] = cum;
      }
      compute_sync();
      if (half == 0) {
        for (int k = 0; k < q; ++k) cum += bars->part[k];
        cd[r] = make_float2(cum, dt);
      }
      if (n + 1 < n_chunks) raw = load_dt(n + 1);
      compute_sync();
      const float2 mine = cd[r];
      const float c_end = cd[kL - 1].x;
      // ---- X' and the skip term's x ----
      if (ok && !mbar_wait(&bars->full[st], (n / C::kStages) & 1, abort_flag)) ok = false;
      ok = __all_sync(0xffffffffu, ok);
      uint32_t xs[kHalf / 2];
      if (ok) {
        const uint8_t* tx = smem + st * C::kStageBytes + 2 * kTileBytes;
        const float w = ex2(c_end - mine.x) * mine.y;
#pragma unroll
        for (int j = 0; j < kHalf; j += 8) {
          const uint32_t o = swz(r, half * kHalf + j);
          const uint4 v = *reinterpret_cast<const uint4*>(tx + o);
          xs[j / 2] = v.x; xs[j / 2 + 1] = v.y; xs[j / 2 + 2] = v.z; xs[j / 2 + 3] = v.w;
          float f[8];
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const float2 u = unpack_bf16x2(xs[j / 2 + k]);
            f[2 * k] = u.x * w;
            f[2 * k + 1] = u.y * w;
          }
          uint4 hi, lo;
          split8(f, hi, lo);
          *reinterpret_cast<uint4*>(xp_hi + o) = hi;
          *reinterpret_cast<uint4*>(xp_lo + o) = lo;
        }
        fence_proxy_async_smem();
      }
      // ---- G -> G * L ----
      if (ok && !mbar_wait(&bars->g_full, n & 1, abort_flag)) {
        if (lane == 0) report_status(a.status, kWaitTmemFullTimeout, 313, h, n);
        ok = false;
      }
      ok = __all_sync(0xffffffffu, ok);
      uint32_t gh[32], gl[32];
      if (ok) {
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const int j0 = half * 64 + c * 32;
          if (j0 <= q * 32 + 31) {   // warp-uniform: some column of the block is at or below the diagonal
            uint32_t v[32];
            tmem_ld_32x32(tmem + kColG + j0 + lane_off, v);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 32; j += 2) {
              const float2 c0 = cd[j0 + j], c1 = cd[j0 + j + 1];
              const float m0 = j0 + j <= r ? __uint_as_float(v[j]) * ex2(mine.x - c0.x) * c0.y : 0.f;
              const float m1 = j0 + j + 1 <= r ? __uint_as_float(v[j + 1]) * ex2(mine.x - c1.x) * c1.y : 0.f;
              const uint32_t hw = pack_bf16x2(m0, m1);
              const float2 f = unpack_bf16x2(hw);
              gh[c * 16 + j / 2] = hw;
              gl[c * 16 + j / 2] = pack_bf16x2(m0 - f.x, m1 - f.y);
            }
          } else {
#pragma unroll
            for (int j = 0; j < 16; ++j) gh[c * 16 + j] = gl[c * 16 + j] = 0u;
          }
        }
        tc_fence_before();
      }
      compute_sync();   // every warp has read its part of G: the region may be overwritten
      if (ok) {
        tc_fence_after();
        tmem_st_32x32(tmem + kColG + half * 32 + lane_off, gh);
        tmem_st_32x32(tmem + kColG + 64 + half * 32 + lane_off, gl);
        tmem_st_wait();
        tc_fence_before();
      }
      mbar_arrive(&bars->m_ready);
      if (ok && !mbar_wait(&bars->y_full, n & 1, abort_flag)) {
        if (lane == 0) report_status(a.status, kWaitTmemFullTimeout, 314, h, n);
        ok = false;
      }
      ok = __all_sync(0xffffffffu, ok);
      if (ok) {
        tc_fence_after();
        const float ei = ex2(mine.x), ee = ex2(c_end);
        const int t = n * kL + r;
        __nv_bfloat16* yo = a.y + static_cast<int64_t>(first + t) * inner + h * P + half * kHalf;
#pragma unroll
        for (int c = 0; c < kHalf; c += 32) {
          uint32_t v[32], u[32];
          tmem_ld_32x32(tmem + kColY + half * kHalf + c + lane_off, v);
          tmem_ld_32x32(tmem + kColYo + half * kHalf + c + lane_off, u);
          tmem_ld_wait();
          if (t < len) {
#pragma unroll
            for (int j = 0; j < 32; j += 8) {
              uint32_t o[4];
#pragma unroll
              for (int k = 0; k < 4; ++k) {
                const float2 x = unpack_bf16x2(xs[(c + j) / 2 + k]);
                const int i = j + 2 * k;
                o[k] = pack_bf16x2(fmaf(dsk, x.x, fmaf(ei, __uint_as_float(u[i]), __uint_as_float(v[i]))),
                                   fmaf(dsk, x.y, fmaf(ei, __uint_as_float(u[i + 1]), __uint_as_float(v[i + 1]))));
              }
              *reinterpret_cast<uint4*>(yo + c + j) = make_uint4(o[0], o[1], o[2], o[3]);
            }
          }
          tmem_ld_32x32(tmem + kColT + half * kHalf + c + lane_off, v);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) S[c + j] = fmaf(S[c + j], ee, __uint_as_float(v[j]));
        }
        tc_fence_before();
      }
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

template <int P>
cudaError_t ssd_launch(const CUtensorMap& m, const SsdArgs& a, cudaStream_t st) {
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(ssd_scan_sm100_kernel<P>, cudaFuncAttributeMaxDynamicSharedMemorySize, SsdCfg<P>::kSmem);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  static_assert(SsdCfg<P>::kSmem <= 227 * 1024, "shared memory");
  static_assert(sizeof(SsdBars) <= 192, "barrier block");
  ssd_scan_sm100_kernel<P><<<dim3(a.s.H, a.sb.n_seq), kThreads, SsdCfg<P>::kSmem, st>>>(m, a);
  return cudaGetLastError();
}

}  // namespace

bool ssd_scan_sm100_ok(const SsdShape& s) {
  return s.N == kN && (s.P == 64 || s.P == 128) && s.G >= 1 && s.H % s.G == 0;
}

cudaError_t launch_ssd_scan_sm100(const SeqBatch& sb, const __nv_bfloat16* xbc, const __nv_bfloat16* dt_raw, int64_t ld_dt,
                                  const float* dt_bias, const float* a_log, const float* d_skip, float* state,
                                  __nv_bfloat16* y, const SsdShape& s, int* status, cudaStream_t st) {
  if (!ssd_scan_sm100_ok(s)) return cudaErrorInvalidValue;
  const uint64_t cols = static_cast<uint64_t>(s.H) * s.P + 2ull * s.G * s.N;
  CUtensorMap m;
  cudaError_t e = encode_tma_2d(&m, xbc, 2, cols, sb.n_tok, cols * 2, 64, kL);
  if (e != cudaSuccess) return e;
  const SsdArgs a{sb, dt_raw, ld_dt, dt_bias, a_log, d_skip, state, y, s, status};
  return s.P == 64 ? ssd_launch<64>(m, a, st) : ssd_launch<128>(m, a, st);
}

}  // namespace b200
