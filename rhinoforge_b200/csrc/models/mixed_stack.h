// Decoder stack whose layers differ: every layer names its own mixer (latent attention with a sliding window, HGRN2 linear
// attention), head sizes and feed-forward, and the stack adds what such designs share: an fp32 residual stream, a token
// shift in front of every mixer and a gated per-token side input behind every layer.  Activations are fp16 / bf16, or fp32
// throughout (dtype 2).  Like rf_stack_* one handle owns the weight pointers and a static arena and enqueues the whole layer
// loop on a stream, so a decode step can be captured into a CUDA graph.
#pragma once
#include <stdint.h>

#include "../rf_api.h"

#ifdef __cplusplus
extern "C" {
#endif

enum RfMixerKind { RF_MIXER_LATENT_ATTENTION = 0, RF_MIXER_HGRN2 = 1 };
enum RfMixedAct { RF_MIXED_ACT_RELU2 = 0 };

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
} RfMixedConfig;

// Padded sizes: per-head sizes and ranks are multiples of 8 / 16 with zero rows behind the true ones.
typedef struct RfMixedLayer {
  int32_t mixer, heads, dim, vdim, vdim_true;
  int32_t rank, rank_true, window;      // latent attention; window <= 0: unlimited
  int32_t expand_hd;                    // 64 / 128 / 256: portions expand K and V to heads of this size (== dim == vdim)
  int32_t inter;                        // 0: the layer has no feed-forward
  int32_t act;                          // RfMixedAct
  float scale;
  int32_t in_dim;                       // rows of w_in: [q | latent] or [q | f | v]
  const float* norm1; const float* norm2; const float* shift;
  float* shift_state;                   // [slots, hidden]
  const void* w_in; const void* w_o; const void* w_up; const void* w_down;
  const float* latent_norm;
  const void* w_absorb;                 // [heads, rank, dim]: query -> latent space
  const void* w_unabsorb;               // [heads, vdim, rank]: latent space -> value
  const void* w_expand;                 // [2 * heads * expand_hd, rank]: keys of all heads, then values
  void* latent_pool;                    // [pages, 16, rank]
  const float* f_bias; const float* lower; const float* head_norm;
  float* rec_state;                     // [slots, heads, dim, vdim]
  const void* side_gate; const void* side_proj; const float* side_norm;
} RfMixedLayer;

// One step: portions of several sequences packed into rows.  The first `short_seqs` sequences (`short_rows` rows) have fewer
// than long_min tokens each, the rest are prefill-sized.  decode = 1: one row per sequence, seq_of_row / q_start / q_len null.
// h_q_len / h_pos0 are HOST arrays [num_seqs] (new tokens and first position), read only for prefill-sized sequences.
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
// Re-point the per-layer state of a layer (binding another cache object); null keeps the pointer.
int rf_mixed_set_state(int64_t h, int32_t layer, void* latent_pool, float* rec_state, float* shift_state);
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
void rf_mixed_struct_sizes(int32_t* out);   // sizeof: config, layer, forward, RfRows, RfStreamNorm, RfLatentAttn, RfHgrn2, RfHeadLinear

#ifdef __cplusplus
}
#endif
