// Decoder stack whose layers differ: every layer names its own mixer (latent attention with a sliding window, a query latent, a
// rotated key part or another layer's cache, HGRN2 linear attention, grouped-head attention with chunks or windows, sinks, distance
// slopes and convolved projections, a selective scan, a gated delta rule), sizes and feed-forward (dense or a mixture of experts), and
// the stack adds what such designs share: an fp32 residual stream, an embedding of token pairs, norms in front of the sublayers, on
// their outputs or both, a factor on those outputs, a token shift in front of every mixer or a convolution in front of every
// sublayer, a gated per-token side input behind every layer and a soft cap of the logits (all optional).  Activations are
// fp16 / bf16, or fp32 throughout (dtype 2).  Like rf_stack_* one handle owns the weight pointers and a static arena and enqueues the whole layer
// loop on a stream, so a decode step can be captured into a CUDA graph.
#pragma once
#include <stdint.h>

#include "../rf_api.h"

#ifdef __cplusplus
extern "C" {
#endif

enum RfMixerKind { RF_MIXER_LATENT_ATTENTION = 0, RF_MIXER_HGRN2 = 1, RF_MIXER_ATTENTION = 2, RF_MIXER_MAMBA1 = 3, RF_MIXER_DELTA = 4 };
// Feed-forwards: relu(up)^2 (experts: silu(gate) * up), clipped gated unit, silu(gate) * up, gelu(up).  Gated: w_up holds gate rows, then up rows.
enum RfMixedAct { RF_MIXED_ACT_RELU2 = 0, RF_MIXED_ACT_CLIPPED_GLU = 1, RF_MIXED_ACT_SWIGLU = 2, RF_MIXED_ACT_GELU = 3 };

typedef struct RfMixedConfig {
  int32_t layers;
  int32_t hidden, hidden_true;   // row length of the stream (multiple of 8) and the width the norms average over
  int32_t vocab, vocab_ld;       // true vocabulary; rows of w_lm and pitch of the logits (multiple of 8)
  int32_t dtype;                 // 0 fp16, 1 bf16, 2 fp32
  int32_t max_tokens, max_seqs, max_seq_len;
  int32_t side_dim;              // columns of a layer's side-input slice, multiple of 8 (0: no side input)
  int64_t side_ld;               // row length of the side table
  float eps;
  int32_t weights_packed;        // linear weights are tile-major images (16-bit dtypes only)
  int32_t long_min;              // portions of at least this many tokens take the prefill forms
  const void* embed;             // [vocab, hidden]
  const void* side_table;        // [vocab, layers * side_dim]
  const float* final_norm;
  const void* w_lm;              // [vocab_ld, hidden]
  float embed_scale;
  int32_t norm_after;            // 0: sublayers read the normalised stream; 1: they read the stream, norms act on their outputs
  float residual_mult;           // factor of the sublayers' outputs (0 counts as 1)
  float logit_softcap;           // logits <- cap * tanh(logits / cap) (0: none)
  const void* pair_table;        // [pair_buckets + 1, hidden]: embedding of (previous token, token), see RfStreamNorm (null: none)
  int64_t pair_mul_prev, pair_mul_cur;
  int32_t pair_buckets;
  int32_t input_taps;            // > 0: convolution of this many taps in front of every sublayer (input_conv of the layers)
} RfMixedConfig;

// Per-sequence memory of a layer; what a layer does not use is null.
typedef struct RfMixedState {
  void* latent_pool;                    // [pages, 16, rank + rot_pad]; with `shares` that of the layer it attends over
  void* k_pool; void* v_pool;           // [pages, kv_heads, 16, head size]
  int64_t pool_pages;
  float* rec_state;                     // HGRN2, delta rule: [slots, heads, dim, vdim]; scan: [slots, inner, states]
  void* conv_state;                     // delta rule: [slots, taps, 2 kv_heads * dim + heads * vdim]; [slots, taps - 1, inner] or [slots, taps - 1, (heads + 2 kv_heads) * dim]
  float* shift_state;                   // [slots, hidden]
  int32_t* last_token;                  // [slots], one array for the whole stack
  void* input_state[2];                 // [slots, input_taps - 1, hidden]: mixer, feed-forward
} RfMixedState;

// Padded sizes: per-head sizes and ranks are multiples of 8 / 16 with zero rows behind the true ones.
typedef struct RfMixedLayer {
  int32_t mixer, heads, dim, vdim, vdim_true;
  int32_t rank, rank_true, window;      // attention: window <= 0: unlimited
  int32_t expand_hd;                    // 64 / 128 / 256: portions expand K and V to heads of this size (== dim == vdim), or 192: values of 128
  int32_t inter;                        // 0: the layer has no feed-forward
  int32_t act;                          // RfMixedAct (clipped GLU: w_up holds gate rows, then up rows)
  float scale;
  int32_t in_dim;                       // rows of w_in: [q | latent], [query latent | latent | rotated part], [q | f | v], [q | k | v | gate],
                                        // [x | z] or [q | k | v | gate | b | a] (b and a padded to multiples of 8 rows)
  int32_t out_dim;                      // columns of w_o
  const float* norm1; const float* norm2; const float* shift;
  const void* w_in; const void* w_o; const void* w_up; const void* w_down;
  const float* latent_norm;
  const void* w_absorb;                 // [heads, rank, plain]: query -> latent space
  const void* w_unabsorb;               // [heads, vdim, rank]: latent space -> value
  const void* w_expand;                 // [heads * (expand_hd + vdim), rank + rot_pad]: keys of all heads (the rotated part copied), then values
  int32_t plain;                        // unrotated dimensions of a query head (multiple of 8); the rotated ones lie behind them
  int32_t q_rank, q_rank_true;          // > 0: queries go through a latent of this size
  int32_t rot, rot_pad;                 // rotated key part that all heads share: size and columns in the cache
  int32_t shares;                       // 1: no latent of its own, latent_pool is another layer's
  const void* w_uq;                     // [heads * dim, q_rank]
  const float* q_latent_norm;
  const float* f_bias; const float* lower; const float* head_norm;
  const void* side_gate; const void* side_proj; const float* side_norm;
  // grouped-head attention: heads of dim == vdim values (true sizes dim_true, vdim_true)
  int32_t kv_heads, dim_true;
  int32_t tensor_core;                  // 1: heads of 64 / 128 / 256 on the tensor-core kernels; 0: attention by row in fp32
  int32_t chunk;                        // > 0: positions see their own chunk of this many positions
  int32_t gated;                        // the input projection holds an output gate behind the values
  int32_t rot_dims, v_role;             // RfVMix
  float v_lambda;
  const float* cos; const float* sin;   // [positions, rot_dims / 2]
  const float* q_norm; const float* k_norm; const float* sink;
  int32_t keep_first;                   // with a window or chunk: first positions that stay visible
  int32_t norm_all;                     // one norm over all query heads and one over all key heads (weights [heads, dim])
  int32_t gate_by_head;                 // with `gated`: one gate number per head
  int32_t conv_taps;                    // > 0: causal convolution of queries, keys and values (conv_w [taps, (heads + 2 kv_heads) * dim])
  const float* slopes;                  // [heads]: what scores lose per token of distance
  const float* rates;                   // [heads], with slopes: ... per unit of ln(1 + rate * distance)
  float growth; int32_t growth_every;   // growth of the queries with their position (RfQkvInsert)
  // selective scan
  int32_t inner, states, dt_rank, taps;
  const float* conv_w; const float* conv_b; const float* a2; const float* d_skip; const float* dt_bias;
  const void* w_x;                      // [dt_rank + 2 * states, inner]
  const void* w_dt; const void* w_dt_rows;   // [inner, dt_rank]: as the linear layers take it, and row-major
  // mixture of experts (experts > 0; inter is an expert's width, w_up and w_down the banks)
  int32_t experts, top, groups, keep, score_fn, norm_topk, shared_inter;
  int32_t bank_inter;                   // inter padded to the bank's granularity (128 in 16 bits)
  float route_scale;
  const void* router; const float* correction; const void* shared_up; const void* shared_down;
  float act_limit, act_alpha, shared_limit;   // constants of the clipped GLU
  int32_t identity;                     // router outputs behind the experts' whose result is the input itself
  const float* norm1b; const float* norm2b;   // norms of the sublayers' outputs besides those of their inputs
  const float* input_conv[2];           // [input_taps, hidden]: mixer, feed-forward
  const float* rate;                    // delta rule: [heads] exp(A_log); convolution in conv_w and taps, dt_bias, head_norm as above
  int32_t shared_gate;                  // the router holds one more row: the logit of the shared expert's weight
  RfMixedState st;
} RfMixedLayer;

// One step: portions of several sequences packed into rows.  The first `short_seqs` sequences (`short_rows` rows) have fewer
// than long_min tokens each, the rest are prefill-sized.  decode = 1: one row per sequence, seq_of_row / q_start / q_len null.
// h_q_len / h_pos0 are HOST arrays [num_seqs] (new tokens and first position); decode steps do not read them.
typedef struct RfMixedForward {
  const int32_t* ids;
  RfRows rows;
  int32_t tokens, short_seqs, short_rows, decode;
  int32_t max_kv;                       // host bound: keys any short row sees before its window
  const int32_t* h_q_len; const int32_t* h_pos0;
  float* taps;                          // optional [layers, tokens, hidden]: the stream after every layer
} RfMixedForward;

int64_t rf_mixed_create(const RfMixedConfig* cfg);
int rf_mixed_destroy(int64_t h);
int rf_mixed_set_layer(int64_t h, int32_t layer, const RfMixedLayer* w);
// Re-point the per-sequence memory of a layer (binding another cache object).
int rf_mixed_set_state(int64_t h, int32_t layer, const RfMixedState* st);
// Re-point the rotation tables of a layer (a longer context).
int rf_mixed_set_rotation(int64_t h, int32_t layer, const float* cos, const float* sin);
// Raise max_seq_len (a larger cache is bound); the arena has to be planned and bound again.
int rf_mixed_set_context(int64_t h, int32_t max_seq_len);
uint64_t rf_mixed_arena_bytes(int64_t h);
int rf_mixed_bind_arena(int64_t h, void* base, uint64_t bytes);
int32_t* rf_mixed_status_ptr(int64_t h);
int rf_mixed_forward(int64_t h, const RfMixedForward* f, rf_stream_t stream);
// Final norm and logits of `rows` rows of the last forward (row_idx on the device, null: rows 0..rows-1); logits
// [rows, vocab_ld] in the activation dtype; out_ids (optional) receives the arg-max.
int rf_mixed_head(int64_t h, const int32_t* row_idx, int32_t rows, int32_t* out_ids, float* out_vals, void* logits,
                  rf_stream_t stream);
void rf_mixed_struct_sizes(int32_t* out);   // sizeof: config, layer, forward, RfRows, RfStreamNorm, RfLatentAttn, RfHgrn2, RfHeadLinear, state, RfAttn, RfQkvInsert,
                                            // RfConvSilu, RfMamba1, RfMoeRouter, RfMoeExperts, RfLatentInsert, RfHeadRotate, RfDelta

#ifdef __cplusplus
}
#endif
