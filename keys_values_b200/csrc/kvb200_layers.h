// C API of libkvb200_layers: kernels of models whose layers are described one by one (latent attention over a
// ring of latents, grouped attention, state-space recurrence, retention, routed experts, token shift, averages over the depth,
// norms). Conventions as in kvb200.h: launches on the given stream, returns KVB_OK or a negative code, dtype 0 = fp32, 1 = bf16;
// nothing synchronises the device.
//
// A pass works on B rows of T tokens (right padded). Row b belongs to the sequence in slot slots[b]; its first
// token has position start[b], and count[b] <= T of its tokens are real. Padding is computed like tokens but never
// reaches a cache or a state.
#pragma once
#include <stdint.h>

#include "kvb200.h"

#ifdef __cplusplus
extern "C" {
#endif

// ---- layer_edge.cu
// First tokens of a layer stack: x = embed[token] (+ bigram row), fp32, written to hist (entry 0 of the depth
// history); then norm and token shift of the first layer as in kvb_layer_edge. bigram may be NULL; gain NULL: no norm.
int kvb_embed_edge(const long long* idx, const int* prev_token, const void* embed, const void* bigram, long long buckets,
                   long long mul_prev, long long mul_cur, float* hist, const float* gain, const float* shift, float* state, void* h,
                   void* hs, const int* slots, const int* start, const int* count, int B, int T, int width, long long vocab, float eps,
                   int dtype, int* status, void* stream);
// Between two layers: X_new = x_in + mix (+ sum_k w[n,k] · expert_out[row[n,k]]); with a depth history (coef not NULL)
// hist[n_hist] = X_new and x_out = sum_{j <= n_hist} coef[j] · X_j, else x_out = X_new. Then, unless gain is NULL,
// h = x_out / rms(x_out) · gain and hs = h + (h_prev − h) · shift (shift NULL: hs not written). state (slots, width):
// h of the last token of every sequence.
int kvb_layer_edge(const float* x_in, const void* mix, const void* expert_out, const int* expert_row, const float* expert_w, int top,
                   long long expert_ld, float* hist, int n_hist, long long hist_stride, const float* coef, float* x_out,
                   const float* gain, const float* shift, float* state, void* h, void* hs, const int* slots, const int* start,
                   const int* count, int B, int T, int width, float eps, int dtype, void* stream);
// rows of x (fp32, rows[i] or i when rows is NULL) divided by their root mean square, times one number
int kvb_scalar_rmsnorm(const float* x, const long long* rows, const float* gain, void* y, long long n, int width, float eps,
                       int dtype, void* stream);
// pos[slot] += count, prev_token[slot] = last token of the row; rows without tokens stay as they are
int kvb_sequence_advance(const long long* idx, int* pos, int* prev_token, const int* slots, const int* count, int B, int T,
                         void* stream);

// ---- norm_edge.cu
// Between two sublayers: s = sub + sum_k expert_w[n, k] · expert_out[expert_row[n, k]] (sub, expert_out NULL: without); x = x_in +
// norm(s) · after (x_in NULL: without; after NULL: s as it is) + embed[idx] + step (each unless NULL); x_out = x (NULL: not stored; may be
// x_in); h = norm(x) · before, or x (before NULL), unless h is NULL. Rows of `width`, x fp32, sub, expert_out, embed and h of `dtype`,
// weights and step fp32. center: layer norm, else RMS norm.
//
// tokens (NULL: the rows are no tokens of a pass): the n rows are T tokens of n / T rows of a pass. table (NULL: none): row start[b] + t is added
// to x. conv_w (taps, width; NULL: none; with T = 1): h becomes sum_k conv_w[k] · (h of the token taps - 1 - k before), zero before a sequence's
// start; conv_ring (slots, taps, width) of `dtype` holds the last h of every sequence, position p in row p mod taps.
typedef struct {
  const int *slots, *start, *count;
  int T, taps;
  const void* table;
  long long table_rows;
  const float* conv_w;
  void* conv_ring;
} kvb_edge_tokens;
int kvb_norm_edge(const float* x_in, const void* sub, const void* expert_out, const int* expert_row, const float* expert_w, int top,
                  long long expert_ld, const float* after, float* x_out, const float* before, void* h, const long long* idx,
                  const void* embed, long long vocab, const float* step, long long n, int width, float eps, int center, int dtype,
                  const kvb_edge_tokens* tokens, int* status, void* stream);

// ---- grouped_attn.cu
// One grouped-query attention. `maps` queries and keys per head over the same values (1, or 2 for differential attention, whose
// result is norm(map 1 - lambda · map 2) · post per head, the norm an RMS norm over vdim without a weight). Rows of the cache
// (slots, len, kv_heads, maps · dimp + vdp) = [keys of the maps | value] of a position; dimp, vdp multiples of 8, padding zero.
// Position i sees j <= i, and only those with i - j < window or j < keep (window > 0), or in i's own part of `chunk` positions (chunk > 0).
// ring > 0: the first `head` positions have rows of their own, position p >= head has row head + (p - head) mod ring (both multiples of
// 128); a pass must not be longer than the ring minus what a position looks back.
// pool > 0 (with a window and a ring, without keep): rows 0 .. head - 1 are blocks, row b the means of keys and values of the positions
// b · pool .. b · pool + pool - 1; position p has row head + p mod ring. A query at position i also sees, in the same softmax, every block that
// ends at i - window or before.
// score = q·k · scale, then softcap · tanh(score / softcap) if softcap > 0. sink: one more term exp(sink_w[head]) in the denominator
// (sink_w NULL: exp(0)). gate_cols: columns of the gate projection per head, 0 (none), 1 or vdp: out *= sigmoid(gate). One map: out *= post.
// out_ld: leading dimension of out, 0: heads · vdp. borrowed: keys and values belong to another layer, prep makes queries only. q_scale: factor
// of every head's queries (NULL: none).
typedef struct {
  int heads, kv_heads, maps, dim, dimp, vdim, vdp;
  int rot_dims, value_col, head_norm;
  int window, keep, chunk;
  int head, ring;
  int sink, gate_cols;
  float scale, softcap;
  float lambda, post, eps;
  int pool, borrowed;
  long long out_ld;
  const float* sink_w;
  const float* q_scale;
} kvb_attention;
// Columns of qkv: queries (heads · maps · dimp), keys (kv_heads · maps · dimp), values from value_col on; value_col = heads · dimp: the
// values are the keys as they are in qkv. RMS norm (norm_q, norm_k NULL: none) over the whole projection with weights of its size, or
// (head_norm) over every head and map with dimp weights. Rotation of the first rot_dims dimensions by position · freq. With pool: the blocks
// whose last position the pass brings get their rows.
int kvb_grouped_prep(const void* qkv, long long ld, const float* norm_q, const float* norm_k, const float* freq, void* q, void* rows,
                     const int* slots, const int* start, const int* count, int B, int T, int len, const kvb_attention* a, int dtype,
                     void* stream);
// Queries (B, T, heads · maps, dimp), the first of row b at position start[b], over the rows of its slot. gate: leading dimension
// gate_ld, NULL: none. out (B, T, out_ld).
int kvb_grouped_attend(const void* q, const void* rows, const void* gate, long long gate_ld, void* out, const int* slots,
                       const int* start, int B, int T, int len, const kvb_attention* a, int dtype, void* stream);

// The same in bf16: several tokens on tcgen05 (latent_sm100.cu), one token per sequence split over the positions.
int kvb_grouped_attend_tc_supported(const kvb_attention* a);
int kvb_grouped_attend_tc(const void* q, const void* rows, const void* gate, long long gate_ld, void* out, const int* slots,
                          const int* start, int B, int T, int n_slots, int len, const kvb_attention* a, int* status, void* stream);
int kvb_grouped_decode_supported(const kvb_attention* a);
long long kvb_grouped_decode_scratch_bytes(int B, int len, const kvb_attention* a);
int kvb_grouped_decode(const void* q, const void* rows, const void* gate, long long gate_ld, void* out, void* scratch, const int* slots,
                       const int* start, int B, int n_slots, int len, const kvb_attention* a, int* status, void* stream);

// ---- ssm.cu
// Columns of u (ld): z (heads · vdp), from `col` on the channels x (heads · vdp) | B (groups · np) | C (groups · np), from
// dt_col on the step sizes (heads). vdp, np multiples of 8. ring (slots, taps, channels), state (slots, heads, np, vdp) fp32.
// The convolution has a bias (NULL: none) and a silu behind it, or (silu 0) nothing.
int kvb_short_conv(const void* u, long long ld, int col, const float* w, const float* bias, void* out, void* ring, const int* slots,
                   const int* start, const int* count, int B, int T, int channels, int taps, int silu, int dtype, void* stream);
int kvb_state_scan(const void* u, long long ld, int dt_col, const void* xbc, const float* dt_bias, const float* a_log,
                   const float* skip, float* state, void* y, const int* slots, const int* start, const int* count, int B, int T,
                   int heads, int groups, int vdp, int np, int dtype, void* stream);
// the same in bf16 on tcgen05 (ssm_sm100.cu), for vdp and np up to 128
int kvb_state_scan_tc_supported(int heads, int groups, int vdp, int np);
long long kvb_state_scan_tc_scratch_bytes(int B, int T, int heads, int groups, int vdp, int np);
int kvb_state_scan_tc(const void* u, long long ld, int dt_col, const void* xbc, const float* dt_bias, const float* a_log,
                      const float* skip, float* state, void* y, void* scratch, const int* slots, const int* start, const int* count,
                      int B, int T, int heads, int groups, int vdp, int np, int* status, void* stream);
int kvb_state_step(const void* u, long long ld, int col, int dt_col, const float* w, const float* bias, const float* dt_bias,
                   const float* a_log, const float* skip, void* ring, float* state, void* y, const int* slots, const int* start,
                   const int* count, int B, int heads, int groups, int vdp, int np, int taps, int dtype, void* stream);
// ---- retention.cu (scans: ssm.cu, ssm_sm100.cu). S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head; state (slots, heads, np, vdp)
// fp32, np = key size and vdp = value size padded to multiples of 8.
// in (n, ld) fp32 = [queries heads · np | keys heads · np] -> out (n, 2 · heads · np): both rotated by position · freq, keys times key_scale
int kvb_retention_prep(const float* in, long long ld, const float* freq, void* out, const int* start, int B, int T, int heads, int np,
                       int rot_dims, float key_scale, int dtype, void* stream);
// qk as prep leaves it, v (ldv) heads · vdp columns; y (B, T, heads · vdp), zero in padding
int kvb_retention_scan(const void* v, long long ldv, const void* qk, long long ldqk, const float* decay, float* state, void* y,
                       const int* slots, const int* start, const int* count, int B, int T, int heads, int vdp, int np, int dtype,
                       void* stream);
// the same in bf16 on tcgen05, sizes and scratch as kvb_state_scan_tc with groups = heads
int kvb_retention_scan_tc(const void* v, long long ldv, const void* qk, long long ldqk, const float* log2_decay, float* state, void* y,
                          void* scratch, const int* slots, const int* start, const int* count, int B, int T, int heads, int vdp, int np,
                          int* status, void* stream);
// out = y / rms(y) · weight · silu(gate) head by head (the norm over vdim columns; weight: vdp numbers, NULL: ones); gate has leading
// dimension ld
int kvb_head_norm_gate(const void* y, const void* gate, long long ld, const float* weight, void* out, long long n, int heads, int vdim, int vdp,
                       float eps, int dtype, void* stream);
// One token per sequence, everything between the projections: u (B, ld) fp32 = [queries | keys | values | gate]; out (B, heads · vdp)
int kvb_retention_step(const float* u, long long ld, const float* freq, const float* decay, float* state, void* out, const int* slots,
                       const int* start, const int* count, int B, int heads, int vdim, int vdp, int np, int rot_dims, float key_scale,
                       float eps, int dtype, void* stream);

// ---- gated_linear.cu (scans: ssm.cu, ssm_sm100.cu). S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t · q_scale per head, with alpha =
// sigmoid(bias + sum_r a_r · w[r])^(inv_tau) a number per token and key channel. in (n, ld) fp32 = [queries heads · np | keys heads · np | a
// (rank)], w (rank, heads · np), bias (heads · np) fp32.
typedef struct {
  const float *in, *w, *bias;
  long long ld;
  int heads, np, rank;
  float inv_tau, q_scale;
} kvb_gated_linear;
// Chunks of 128 tokens: out (B, T, 2 heads · np) bf16 = queries times the decay since the middle of their chunk and keys over the same;
// factor (B, chunks, heads, np, 2): log2 of the decays of a chunk's first and second half. far[b, head] = 1 where these leave the range in which
// such products are exact (the scan skips that head; the plain one takes it). Padding becomes zero.
int kvb_gated_linear_prep(const kvb_gated_linear* g, void* out, float* factor, int* far, const int* count, int B, int T, void* stream);
// v (ldv) heads · vdp columns; y (B, T, heads · vdp), zero in padding. only (NULL: all): heads of rows where it is 0 are left alone.
int kvb_gated_linear_scan(const kvb_gated_linear* g, const void* v, long long ldv, float* state, void* y, const int* only, const int* slots,
                          const int* start, const int* count, int B, int T, int vdp, int dtype, void* stream);
// the same in bf16 on tcgen05 from what prep left; sizes as kvb_state_scan_tc with groups = heads
long long kvb_gated_linear_scan_tc_scratch_bytes(int B, int T, int heads, int vdp, int np);
int kvb_gated_linear_scan_tc(const void* v, long long ldv, const void* qk, const float* factor, const int* far, float* state, void* y,
                             void* scratch, const int* slots, const int* start, const int* count, int B, int T, int heads, int vdp, int np,
                             int* status, void* stream);
// One token per sequence, everything between the projections: in = [queries | keys | a | values from v_col on | gate]; norm weight (vdp); out
// (B, heads · vdp)
int kvb_gated_linear_step(const kvb_gated_linear* g, int v_col, const float* norm, float* state, void* out, const int* slots, const int* start,
                          const int* count, int B, int vdim, int vdp, float eps, int dtype, void* stream);

// ---- gated_recurrence.cu. Channels in `blocks` parts of pp (a multiple of 8). S_t = a S_(t-1) + sqrt(1 - a^2) i x with log2 a = rate · r, r =
// sigmoid(zr + bias_r), i = sigmoid(zi + bias_i); state (slots, channels) fp32.
typedef struct {
  const float *conv, *conv_bias, *bias_r, *bias_i, *rate;  // conv (taps, channels), others (channels)
  const void* gates;                                       // (blocks, pp, 2 pp): x of a part times this = zr | zi
  int blocks, pp, taps;
  float scale;
} kvb_gated_recurrence;
// x (B, T, channels) behind its convolution, z (blocks, B · T, 2 pp) fp32, y (ldy) channels; out (ldo) = S · gelu(y) · scale, zero in padding
int kvb_gated_recurrence_scan(const kvb_gated_recurrence* g, const void* x, const float* z, const void* y, long long ldy, float* state, void* out,
                              long long ldo, const int* slots, const int* start, const int* count, int B, int T, int dtype, int* status, void* stream);
// One token per sequence, convolution and gates included: u (ld) = [y: channels | x: channels]; ring (slots, taps, channels)
int kvb_gated_recurrence_step(const kvb_gated_recurrence* g, const void* u, long long ld, void* ring, float* state, void* out, long long ldo,
                              const int* slots, const int* start, const int* count, int B, int dtype, void* stream);

// ---- ssm.cu
// out = norm(y · silu(z)) · weight in `parts` equal parts of the heads · vdim unpadded columns
int kvb_gated_group_norm(const void* y, const void* z, long long ld, const float* weight, void* out, long long n, int heads,
                         int vdim, int vdp, int parts, float eps, int dtype, void* stream);
// act 1: x = relu(x)^2 in place
int kvb_activate(void* x, long long n, int act, int dtype, void* stream);

// ---- latent_attn.cu
// One row of the latent storage: [c (kv_rank, padded to kvp) | rotated key part (rot, padded to rp)], kvp and rp
// multiples of 8, padding zero. Queries: [unrotated (dim padded to dimp) | rotated (rot padded to rp)] per head.
// prep: latent rows go to latent (B, P+T, kvp+rp) from row P on (NULL: not) and those of the last ring_len real tokens to ring
// (slots, ring_len, kvp+rp) (NULL: not), position p in row p mod ring_len.
int kvb_latent_prep(const void* qkv, long long ld, const float* norm_w, const float* freq, void* q, void* latent, void* ring,
                    const int* slots, const int* start, const int* count, int B, int T, int P, int ring_len, int heads, int dim,
                    int dimp, int rot, int rot_dims, int rp, int kv_rank, int kvp, float eps, int dtype, void* stream);
// latent[b, j] (j < P) = ring row of position start[b] − P + j, zero where there is none
int kvb_ring_gather(const void* ring, void* latent, const int* slots, const int* start, int B, int T, int P, int ring_len, int lw,
                    int dtype, void* stream);
// Attention of T new tokens over P + T expanded keys: kv (B, P+T, heads, dimp + vdp) = [unrotated key | value],
// latent (B, P+T, lw) holds the rotated key part at column kvp. out (B, T, heads, vdp).
int kvb_latent_attend(const void* q, const void* kv, const void* latent, void* out, const int* start, int B, int T, int P, int heads,
                      int dimp, int rp, int kvp, int vdp, int window, float scale, int dtype, void* stream);
// One new token per sequence over its ring, in latent space: q_abs (heads, B, kvp) = W_uk^T q, q (B, heads, dimp + rp) for
// the rotated part, out (heads, B, kvp) = weighted latents.
long long kvb_latent_decode_scratch_bytes(int B, int heads, int kvp, int rp, int ring_len);
int kvb_latent_decode(const void* q_abs, const void* q, const void* ring, void* out, void* scratch, const int* slots,
                      const int* start, int B, int n_slots, int heads, int dimp, int rp, int kvp, int ring_len, float scale,
                      int dtype, int simple, int* status, void* stream);

// ---- latent_sm100.cu: kvb_latent_attend for bf16 on tcgen05
int kvb_latent_attend_tc_supported(int dimp, int rp, int vdp);
int kvb_latent_attend_tc(const void* q, const void* kv, const void* latent, void* out, const int* start, int B, int T, int P,
                         int heads, int dimp, int rp, int kvp, int vdp, int window, float scale, int* status, void* stream);

// ---- moe.cu
// Router. score 0: softmax over the experts' fp32 logits, 1: sigmoid of each. correction (n_expert, NULL: none) is added for the choice
// only. groups > 1: equal groups of neighbouring experts, a group's score is the sum of its two largest choice scores, and only experts
// of the `keep` best groups can be chosen. renormalize: the chosen scores are divided by their sum + eps.
typedef struct {
  int score, groups, keep, renormalize;
  float eps;
  const float* correction;
} kvb_router;
// The `top` experts with the largest choice scores (ties: lower index first), their scores in weight (n, top) fp32. Every choice gets a
// row of the buffer sorted by expert: the rows of an expert start at a multiple of `tile`; row (n, top), tile_expert / tile_row (one
// entry per tile in use), plan[0] = number of tiles. counters: n_expert ints of scratch.
int kvb_moe_route(const float* logits, int* expert, float* weight, int* row, int* counters, int* plan, int* tile_expert,
                  int* tile_row, long long n, int n_expert, int top, int tile, int max_tiles, const kvb_router* router, void* stream);
// sorted[row[n, k]] = h[n] (columns beyond width zero up to ld)
int kvb_moe_gather(const void* h, const int* row, void* sorted, long long n, int top, int width, long long ld, int dtype, void* stream);
// out[r] = act(w[expert of r's tile] · in[r]) for all rows of the tiles in use; in (rows, ldk), w (n_expert, n_out, ldk),
// out (rows, ldo) with columns n_out .. ldo zero. act 0: none, 1: square of relu, 2: gated unit, rows 2 f and 2 f + 1 of w are gate and up
// projection of result f (n_out counts both, out has half as many columns).
int kvb_moe_gemm(const void* in, const void* w, void* out, const int* plan, const int* tile_expert, const int* tile_row, int tile,
                 int max_tiles, int n_expert, int n_out, int k, long long ldk, long long ldo, int act, int dtype, int simple,
                 int* status, void* stream);

// out (n, ldo) = silu(x[:, :ff]) · x[:, up : up + ff], zero from column ff on. limit > 0: g · sigmoid(1.702 g) · (u + 1) instead, with g = the
// first factor's input, at most limit, and u = the second one, within ± limit
int kvb_glu(const void* x, void* out, long long n, long long ldx, int up, int ff, int ldo, float limit, int dtype, void* stream);

#ifdef __cplusplus
}
#endif
