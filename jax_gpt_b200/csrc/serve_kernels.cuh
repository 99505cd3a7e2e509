// Serving kernels shared by packed (ragged) batches: embeddings with a bigram table, norms of a 32-bit residual,
// few-row linear layers, latent attention over paged rows, table-routed experts (see serve_kernels.cu), and the
// state-space layers (see ssm_kernels.cu, ssd_scan_sm100.cu). Activations are fp32 or bf16 (`f32`); residuals,
// scores, norms and recurrent states are fp32 in both.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace b200 {

// One step's tokens, packed: sequence b owns rows cu[b] .. cu[b+1]-1, its first row sits at position start[b].
struct SeqBatch {
  const int* ids;      // [n_seq] cache slot of every sequence
  const int* cu;       // [n_seq + 1]
  const int* tok_seq;  // [n_tok] sequence of every row
  const int* start;    // [n_seq]
  int n_seq, n_tok;
};

// start[b] = lens[slot]; lens[slot] += tokens of b; prev_tok[b] = prev[slot]; prev[slot] = last token of b.
cudaError_t launch_seq_begin(const int* ids, const int* cu, const int* tokens, int n_seq, int max_slots, int* lens,
                             int* prev, int* start, int* prev_tok, int* status, cudaStream_t st);

// x[n, :] = embed[token] (+ bigram[row], row = (previous * mul_prev + token * mul_cur) mod buckets, or `buckets`
// for a sequence's first token). x is fp32.
cudaError_t launch_embed_bigram(bool f32, const SeqBatch& sb, const int* tokens, const int* prev_tok, const void* embed,
                                int vocab, const void* bigram, long long buckets, long long mul_prev, long long mul_cur,
                                int D, float* x, int* status, cudaStream_t st);

// out[r, :] = layer norm (mode 0, gamma and beta) or RMS norm (mode 1, gamma) of the fp32 row r.
cudaError_t launch_norm_rows(bool f32_out, int mode, const float* x, const float* gamma, const float* beta, void* out,
                             int rows, int D, float eps, cudaStream_t st);

enum RowAct : int { kActNone = 0, kActRelu2 = 1 };
// y[m, n] = act(sum_k x[m, k] w[n, k]); out_mode 0: activation dtype, 1: fp32, 2: added to fp32 y. Few rows.
cudaError_t launch_rows_linear(bool f32, const void* x, int64_t ldx, const void* w, int64_t ldw, void* y, int64_t ldy,
                               int M, int N, int K, int act, int out_mode, cudaStream_t st);

struct RopeTable {
  const float* cos;    // [max_pos, dims / 2], amplitude folded in
  const float* sin;
  int max_pos, dims;   // the first `dims` features turn in interleaved pairs (2i, 2i + 1)
};
struct PagedRows {
  void* pool;               // one layer: [n_pages, page_size, width], activation dtype
  const int* block_table;   // [max_slots, max_pages]
  int page_size, max_pages, n_pages, width;
};

// y [n_tok, ldy] = [down-projected query: q_rank | compressed kv: R | rotary key: dr]. cq = RMS norm of the first
// part; the token's cache row becomes [RMS norm of the second | rotated third], also written to lat [n_tok, R + dr]
// when that is not null.
cudaError_t launch_mla_prepare(bool f32, const SeqBatch& sb, const void* y, int64_t ldy, int q_rank, int R, int dr,
                               const float* q_gamma, const float* kv_gamma, float eps, const RopeTable& rope,
                               const PagedRows& pages, void* cq, void* lat, int* status, cudaStream_t st);

// Decompressed prefill operands: rotates the last dr features of every query head in place (q [n_tok, H, dn + dr])
// and writes k [n_tok, H, dn + dr] = [kn | lat[:, R:]].
cudaError_t launch_mla_rope_qk(bool f32, const SeqBatch& sb, void* q, const void* kn, int64_t ldkn, const void* lat,
                               int64_t ldlat, int R, void* k, int H, int dn, int dr, const RopeTable& rope, cudaStream_t st);

// qf [n_tok, H, R + dr] = [q_nope W_uk | rotated q_rope] with w_uk [H * dn, R].
cudaError_t launch_mla_absorb_q(bool f32, const SeqBatch& sb, const void* q, const void* w_uk, void* qf, int H, int dn,
                                int dr, int R, const RopeTable& rope, cudaStream_t st);
// o [n_tok, H * dv] = o_lat [n_tok, H, R] W_uv with w_uv [H * dv, R].
cudaError_t launch_mla_absorb_out(bool f32, const void* o_lat, const void* w_uv, void* o, int n_tok, int H, int dv, int R,
                                  cudaStream_t st);

// Causal softmax attention of qf over the pages: row n attends to positions 0 .. pos(n) of its sequence; values are
// the first R features of a cached row; `sink` (optional, [H]) adds exp(sink) to every denominator. n_splits > 1
// cuts the keys into ranges merged by a second kernel (part_o [n_tok, H, S, R], part_ml [n_tok, H, S, 2] fp32).
cudaError_t launch_latent_attention(bool f32, const SeqBatch& sb, const void* qf, const PagedRows& pages, int R,
                                    const float* sink, float scale, int H, int n_splits, float* part_o, float* part_ml,
                                    void* o_lat, cudaStream_t st);

// Experts chosen by a table over token ids (experts of token t: table[t, :top], each with weight 1 / top).
struct GluArgs {
  float limit, alpha;  // g = min(gate, limit), u = clamp(up, -limit, limit): g * sigmoid(alpha * g) * (u + 1)
};
cudaError_t launch_table_experts_up(bool f32, const void* x, const int* tokens, const int* table, int vocab, int top, int E,
                                    const void* w_gate_up, GluArgs glu, void* h, int M, int D, int I, int* status,
                                    cudaStream_t st);
cudaError_t launch_table_experts_down(bool f32, const void* h, const int* tokens, const int* table, int vocab, int top,
                                      int E, const void* w_down, float* x, int M, int D, int I, cudaStream_t st);
// Grouped path: rows of expert e start at offs[e]; pair p = (token, choice) sits in row offs[idx[p]] + pos[p].
cudaError_t launch_moe_gather_rows(const __nv_bfloat16* x, const int* idx, const int* pos, const int* offs_end,
                                   const int* counts, int top, __nv_bfloat16* xs, int* row_of, int M, int D, cudaStream_t st);
cudaError_t launch_clamped_glu(const __nv_bfloat16* gu, GluArgs glu, __nv_bfloat16* h, int rows, int I, cudaStream_t st);
cudaError_t launch_moe_combine_rows(const __nv_bfloat16* ys, const int* row_of, int top, float w, float* x, int M, int D,
                                    cudaStream_t st);

// ---- state-space layers ------------------------------------------------------------------------------------------
// Causal depthwise convolution of packed rows with bias and SiLU. ring [slots, taps, C] fp32 holds the raw input of
// position p in row p % taps; rows of the positions before `start` are read from it, the portion's last taps - 1
// inputs are stored afterwards.
cudaError_t launch_ssm_conv(bool f32, const SeqBatch& sb, const void* x, int64_t ldx, const float* w, const float* bias,
                            float* ring, void* y, int C, int taps, cudaStream_t st);

struct SsdShape {
  int H, P, N, G;      // heads, head width, state size, groups of B / C
};
// y[n, h*P + p] = C . S + D x with S_t = exp(-exp(A_log) dt) S + dt B x^T, dt = softplus(dt_raw + dt_bias);
// xbc [n_tok, H*P + 2 G N] = [x | B | C]; state [slots, H, N, P] fp32 (ignored where start == 0, always written).
cudaError_t launch_ssd_scan(bool f32, const SeqBatch& sb, const void* xbc, const void* dt_raw, int64_t ld_dt,
                            const float* dt_bias, const float* a_log, const float* d_skip, float* state, void* y,
                            const SsdShape& s, cudaStream_t st);
// The same on tensor cores, 128-token chunks: bf16, N = 128, P a multiple of 64.
bool ssd_scan_sm100_ok(const SsdShape& s);
cudaError_t launch_ssd_scan_sm100(const SeqBatch& sb, const __nv_bfloat16* xbc, const __nv_bfloat16* dt_raw, int64_t ld_dt,
                                  const float* dt_bias, const float* a_log, const float* d_skip, float* state,
                                  __nv_bfloat16* y, const SsdShape& s, int* status, cudaStream_t st);

// One token per sequence: convolution window, step sizes, state update, skip and gate in one launch.
// zxd [n_seq, ldz] = [z | x | B | C | dt]; y [n_seq, H*P] fp32 = (S^T C + D x) silu(z).
cudaError_t launch_ssm_decode(bool f32, const SeqBatch& sb, const void* zxd, int64_t ldz, const float* w, const float* bias,
                              float* ring, int taps, const float* dt_bias, const float* a_log, const float* d_skip,
                              float* state, float* y, const SsdShape& s, cudaStream_t st);
// out = RMS norm over `parts` equal pieces of (y silu(z)) times gamma; z null: y is gated already. y fp32 (y_f32) or
// activation dtype.
cudaError_t launch_gated_group_norm(bool f32, bool y_f32, const void* y, const void* z, int64_t ldz, const float* gamma,
                                    void* out, int rows, int D, int parts, float eps, cudaStream_t st);

}  // namespace b200
