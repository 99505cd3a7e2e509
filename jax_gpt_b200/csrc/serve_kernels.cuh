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

// x[r, :] = (add ? x[r, :] : 0) + rms(y[r, :]) gpost; out[r, :] = rms(x[r, :]) gnext unless out is null. x fp32, y fp32
// (y_f32) or bf16.
cudaError_t launch_residual_norm(bool y_f32, bool f32_out, const void* y, const float* gpost, float* x, bool add,
                                 const float* gnext, void* out, int rows, int D, float eps, cudaStream_t st);

// kActXielu: a z^2 + z / 2 for z > 0, b (exp(z) - 1 - z) + z / 2 otherwise
enum RowAct : int { kActNone = 0, kActRelu2 = 1, kActSilu = 2, kActSiluGlu = 3, kActXielu = 4 };
struct RowsOut {
  void* y;             // [M, ldy]
  int64_t ldy;
  int act;             // kActSiluGlu: w holds 2 N rows, y = silu(gate) * up
  int out_mode;        // 0: activation dtype, 1: fp32, 2: added to fp32 y
  float* y2;           // features n >= n1 go to y2[m, n - n1] in fp32, without the activation (n1 = N: none do)
  int64_t ldy2;
  int n1;
  float act_a, act_b;  // kActXielu
};
// y[m, n] = act(sum_k x[m, k] w[n, k]). Few rows.
cudaError_t launch_rows_linear(bool f32, const void* x, int64_t ldx, const void* w, int64_t ldw, int M, int N, int K,
                               const RowsOut& out, cudaStream_t st);

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

// y [n_tok, ldy] = [down-projected query: q_rank (may be 0) | compressed kv: R | rotary key: dr]. cq = RMS norm of the first
// part; the token's cache row becomes [RMS norm of the second | rotated third], also written to lat [n_tok, R + dr]
// when that is not null.
cudaError_t launch_mla_prepare(bool f32, const SeqBatch& sb, const void* y, int64_t ldy, int q_rank, int R, int dr,
                               const float* q_gamma, const float* kv_gamma, float eps, const RopeTable& rope,
                               const PagedRows& pages, void* cq, void* lat, int* status, cudaStream_t st);

// Decompressed prefill operands: rotates the last dr features of every query head in place (q [n_tok, H, dn + dr])
// and writes k [n_tok, H, dn + dr] = [kn | lat[:, R:]].
cudaError_t launch_mla_rope_qk(bool f32, const SeqBatch& sb, void* q, int64_t ldq, const void* kn, int64_t ldkn, const void* lat,
                               int64_t ldlat, int R, void* k, int H, int dn, int dr, const RopeTable& rope, cudaStream_t st);

// qf [n_tok, H, R + dr] = [q_nope W_uk | rotated q_rope] with w_uk [H * dn, R]; rows of q are ldq apart.
cudaError_t launch_mla_absorb_q(bool f32, const SeqBatch& sb, const void* q, int64_t ldq, const void* w_uk, void* qf, int H, int dn,
                                int dr, int R, const RopeTable& rope, cudaStream_t st);
// o [n_tok, H * dv] = o_lat [n_tok, H, R] W_uv with w_uv [H * dv, R], times sigmoid(gate [n_tok, ldg]) unless that is null.
cudaError_t launch_mla_absorb_out(bool f32, const void* o_lat, const void* w_uv, const void* gate, int64_t ldg, void* o, int n_tok, int H,
                                  int dv, int R, cudaStream_t st);
// o [rows, N] *= sigmoid(gate [rows, ldg]) in place.
cudaError_t launch_sigmoid_gate(bool f32, void* o, const void* gate, int64_t ldg, int rows, int N, cudaStream_t st);

// Causal softmax attention of qf over the pages: row n attends to the last `window` positions up to pos(n) of its sequence; values are
// the first R features of a cached row; `sink` (optional, [H]) adds exp(sink) to every denominator. n_splits > 1
// cuts the keys into ranges merged by a second kernel (part_o [n_tok, H, S, R], part_ml [n_tok, H, S, 2] fp32).
cudaError_t launch_latent_attention(bool f32, const SeqBatch& sb, const void* qf, const PagedRows& pages, int R,
                                    const float* sink, float scale, int window, int H, int n_splits, float* part_o, float* part_ml,
                                    void* o_lat, cudaStream_t st);

// Experts of a token: table[token, :top] (each with weight 1 / top), or with `logits` [M, E] fp32 the `top` largest, whose
// sigmoid scores multiply the expert's input.
struct ExpertChoice {
  const int* tokens;
  const int* table;
  int vocab;
  const float* logits;
  int top, E;
};
struct GluArgs {
  float limit, alpha, shift;  // g = min(gate, limit), u = clamp(up, -limit, limit): g * sigmoid(alpha * g) * (u + shift)
};
// h[m * top + j] = glu of the token's j-th expert; x[m] += out_scale * sum of the experts' outputs.
cudaError_t launch_experts_up(bool f32, const void* x, const ExpertChoice& c, const void* w_gate_up, GluArgs glu, void* h, int M,
                              int D, int I, int* status, cudaStream_t st);
cudaError_t launch_experts_down(bool f32, const void* h, const ExpertChoice& c, const void* w_down, float out_scale, float* x,
                                int M, int D, int I, cudaStream_t st);
cudaError_t launch_sigmoid_topk(const ExpertChoice& c, int M, int* ids, float* weights, int* status, cudaStream_t st);
// Grouped path: rows of expert e start at offs[e]; pair p = (token, choice) sits in row offs[idx[p]] + pos[p]. w_pair
// (optional) travels to w_row by the same permutation and scales gate and up before the activation.
cudaError_t launch_moe_gather_rows(const __nv_bfloat16* x, const int* idx, const int* pos, const int* offs_end,
                                   const int* counts, const float* w_pair, int top, __nv_bfloat16* xs, int* row_of, float* w_row,
                                   int M, int D, cudaStream_t st);
cudaError_t launch_clamped_glu(const __nv_bfloat16* gu, const float* w_row, GluArgs glu, __nv_bfloat16* h, int rows, int I,
                               cudaStream_t st);
cudaError_t launch_moe_combine_rows(const __nv_bfloat16* ys, const int* row_of, int top, float w, float* x, int M, int D,
                                    cudaStream_t st);

// ---- windowed attention (window_attention.cu) ------------------------------------------------------------------------
struct WindowMask {
  int size, keep_first;   // i sees j when j <= i and (i - j < size or j < keep_first); no window: size 1 << 30
  int pool;               // > 0 (then keep_first 0): i also sees the mean of every block of `pool` tokens that lies wholly before its window
};
struct ScoreArgs {
  float scale;
  float softcap;          // > 0: scores become softcap * tanh(score / softcap)
  const float* sink;      // optional [H]: exp(sink) joins the denominator, no key and no value
};
// y [n_tok, ldy] = [q of H heads | k of G heads], D wide. q [n_tok, H, D] = unit RMS norm of the rotated (y + bias); the
// cache row becomes [k likewise | k as projected, the values]; both also go to k, v [n_tok, G, D] unless null. `rope` holds
// half-split pairs (i, i + dims / 2) here.
cudaError_t launch_qk_prepare(bool f32, const SeqBatch& sb, const void* y, int64_t ldy, const float* bias, int H, int G, int D,
                              bool unit_norm, float eps, const RopeTable& rope, const PagedRows& pages, void* q, void* k, void* v,
                              int* status, cudaStream_t st);
// Softmax attention of q [n_tok, H, D] over the pages' rows [K (G D) | V (G DV)] of G kv heads, any sizes; `pooled` [n_pages,
// ceil(page_size / pool), width] holds the block means. n_splits > 1 cuts the visible keys into ranges merged by a second kernel
// (part_o [n_tok, H, S, DV], part_ml [n_tok, H, S, 2] fp32).
cudaError_t launch_window_attention(bool f32, const SeqBatch& sb, const void* q, const PagedRows& pages, const void* pooled, int H, int G,
                                    int D, int DV, WindowMask mask, const ScoreArgs& score, int n_splits, float* part_o, float* part_ml,
                                    void* out, cudaStream_t st);

// ---- interleaved rotation, rotated values (rotated_kv.cu) ----------------------------------------------------------------
// Columns of a projection row and their biases ([heads * width] fp32 or null).
struct QkvRows {
  const void* y;
  int64_t ld;
  int q, k, v;
  const float *bq, *bk, *bv;
};
// q, k turned by `rope`, v by `vrope` (interleaved pairs) into the cache row [K (G dk) | V (G dv)], q [n_tok, H, dkp] and, unless
// null, k [n_tok, G, dkp], v [n_tok, G, dvp]; features past dk / dv are zero there.
cudaError_t launch_qkv_rotate(bool f32, const SeqBatch& sb, const QkvRows& in, const RopeTable& rope, const RopeTable& vrope,
                              const PagedRows& pages, int H, int G, int dk, int dv, int dkp, int dvp, void* q, void* k, void* v, int* status,
                              cudaStream_t st);
// out[n, h * dv + c] = scale sigmoid(g[n, h]) (o [n_tok, H, ldh] turned back by the row's position).
cudaError_t launch_turn_back_gate(bool f32, const SeqBatch& sb, const void* o, int ldh, const void* g, int64_t ldg, const RopeTable& vrope,
                                  float scale, int H, int dv, void* out, int64_t ldo, cudaStream_t st);

// ---- grouped-query operands with mixed values and block means (mixed_kv.cu) ------------------------------------------------
struct MixedKv {
  QkvRows in;              // biases unused
  const float* q_factor;   // optional [n_pos]: q is multiplied by the factor of its position
  int n_pos;
  const void* v_first;     // optional [n_tok, ld_first]: v becomes (1 - lambda) v + lambda v_first
  int64_t ld_first;
  float lambda;
  int H, G, dk, dv;
  int dkp, dvp;            // widths of the dense operands, features past dk / dv are zero
  void* pooled;            // optional [n_pages, ceil(page_size / pool), width]: means of whole blocks of `pool` cache rows
  int pool;
  const int* row0;         // optional [n_seq]: row of a sequence's first token in dense k, v (null: its packed row)
};
// q [n_tok, H, dkp], the cache row [K (G dk) | V (G dv)] and, unless null, dense k [rows, G, dkp], v [rows, G, dvp]. With one token per
// sequence the mean of a block is written with its last row; otherwise launch_pool_rows follows.
cudaError_t launch_mixed_kv(bool f32, const SeqBatch& sb, const MixedKv& a, const PagedRows& pages, void* q, void* k, void* v, int* status,
                            cudaStream_t st);
// Means of the blocks that the step's rows complete. With `pad` [n_seq] they also go to the pad[b] dense rows before row0[b] (zeros
// past the whole blocks); n_rows bounds the work: blocks, or blocks and dense rows, over all sequences.
cudaError_t launch_pool_rows(bool f32, const SeqBatch& sb, const MixedKv& a, const PagedRows& pages, const int* pad, int n_rows, void* k,
                             void* v, int* status, cudaStream_t st);

// ---- residual streams and row activations (stream_kernels.cu) ------------------------------------------------------------
constexpr int kMaxStreams = 16;
struct StreamNorm {
  float* xs;             // [rows, S, D] streams, updated in place
  const float* bias;     // optional [D], added to y
  const float* mix;      // [S, S] indexed [from, to]; null: the streams start with y
  const float* w_out;    // [S] weight of y in every stream
  const float* w_in;     // [S] weights of the streams in u
  const float* gamma;    // [D]
  float* u;              // optional [rows, D]: the combination before its norm
  int rows, S, D, groups;
  float eps;
};
// Streams of the sublayer output y [rows, D] and h = group norm of the next sublayer's input (null: none). y fp32 (y_f32) or bf16.
cudaError_t launch_stream_norm(bool y_f32, bool f32_out, const void* y, const StreamNorm& a, void* h, cudaStream_t st);
// out = c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3 over rows of N features; coef [4].
cudaError_t launch_poly_norm(bool f32, const void* z, int64_t ldz, const float* coef, void* out, int rows, int N, float eps, cudaStream_t st);

// ---- gated linear recurrent unit (gated_lru.cu) ----------------------------------------------------------------------------
struct LruArgs {
  int W, blocks, taps;
  const void* x;           // [n_tok, ldx] convolution input before its bias
  int64_t ldx;
  const float *x_bias, *conv, *conv_bias;   // [W], [W, taps] (current token last), [W]
  float* ring;             // [slots, taps, W]: input of position p in row p % taps
  const void* gates;       // [blocks, 2, W / blocks, W / blocks] = recurrence and input gate, (out, in)
  const float* gates_bias; // [blocks, 2, W / blocks]
  const float* decay;      // [W]: log a = -decay * gate
  float* state;            // [slots, W], ignored where start == 0, always written
  const void* y;           // [n_tok, ldy] output branch before bias and gelu
  int64_t ldy;
  const float* y_bias;     // [W]
  float scale;
  void* out;               // [n_tok, ldo]
  int64_t ldo;
};
// scratch: gated_lru_scratch floats (8-byte aligned), or null for one token per sequence.
int64_t gated_lru_scratch(bool f32, const SeqBatch& sb, const LruArgs& a);
cudaError_t launch_gated_lru(bool f32, const SeqBatch& sb, const LruArgs& a, float* scratch, cudaStream_t st);

// ---- linear attention with a matrix state (linear_attention.cu, ssd_scan_sm100.cu) ---------------------------------------
struct LinShape {
  int H, N, P;            // heads, key width, value width; a row of qkv is [q (H N) | k (H N) | v (H P)]
  float q_scale;
  int silu;               // 1: q, k, v still need their SiLU
};
struct LinGates {
  const float* decay;     // [H] fixed decay per head, or with `raw` set exponential gates:
  const float* raw;       // [n_tok, ld] = [i (H) | f (H)] before bias and cap
  int64_t ld;
  const float* bias;      // [2 H]
  float cap;
  const float* vec;       // [slots, H, N + 1] = [n | m] at the start of the step
  float* vec_new;         // [n_seq, H, N + 1] after it
  float* den;             // [n_tok, H, 4] = {n . q, second part of n . q, exp(-m), -}
  // or with `low` set a decay per key channel, alpha = sigmoid(w2 low + bias2)^(inv_tau):
  const void* low;        // [n_tok, ld_low], R wide, activation dtype
  int64_t ld_low;
  const void* w2;         // [H N, R], activation dtype
  const float* bias2;     // [H N]
  int R;
  float inv_tau;
};
// state [slots, H, N, P] fp32 (ignored where start == 0, always written); y [n_tok, H P] fp32: the numerators.
cudaError_t launch_linear_scan(bool f32, const SeqBatch& sb, const void* qkv, int64_t ld, const LinGates& g, float* state, float* y,
                               const LinShape& s, cudaStream_t st);
// One token per sequence.
cudaError_t launch_linear_step(bool f32, const SeqBatch& sb, const void* qkv, int64_t ld, const LinGates& g, float* state, float* y,
                               const LinShape& s, cudaStream_t st);
// Chunked on tensor cores: bf16, N = 128, P a multiple of 64, q_scale > 0, activations applied. y bf16.
bool linear_scan_sm100_ok(const LinShape& s);
cudaError_t launch_linear_scan_sm100(const SeqBatch& sb, const __nv_bfloat16* qkv, int64_t ld, const LinGates& g, float* state,
                                     __nv_bfloat16* y, const LinShape& s, int* status, cudaStream_t st);
// Decays per key channel, chunked on tensor cores (gla_chunk.cu): bf16, N a multiple of 16 up to 128, P and ld multiples of 8, R <= 64,
// activations applied. scratch: gla_chunked_scratch bytes. y bf16.
bool gla_chunked_ok(const LinShape& s, int64_t ld, int R);
int64_t gla_chunked_scratch(const SeqBatch& sb, const LinShape& s);
cudaError_t launch_gla_chunked(const SeqBatch& sb, const __nv_bfloat16* qkv, int64_t ld, const LinGates& g, float* state, __nv_bfloat16* y,
                               const LinShape& s, void* scratch, cudaStream_t st);
struct HeadNorm {
  int parts;
  float eps, den_eps;
  const float* den;       // optional, with pieces = heads: y is divided by max(|n . q|, exp(-m)) + den_eps first
  const float* vec_new;   // optional: copied to vec at the slot of the sequence, by the last row of every sequence
  float* vec;
  int vec_len;
  int gate;               // 0: sigmoid(z), 1: silu(z)
};
// out = RMS norm over `parts` equal pieces of y, times gamma and the gate of z. y fp32 (y_f32) or activation dtype.
cudaError_t launch_head_norm_gate(bool f32, bool y_f32, const SeqBatch& sb, const void* y, const void* z, int64_t ldz,
                                  const float* gamma, void* out, int D, const HeadNorm& a, cudaStream_t st);

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
