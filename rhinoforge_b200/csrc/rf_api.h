// C ABI of librf_b200: every entry point takes raw device pointers and a CUDA
// stream, allocates nothing unless its comment says so, and returns 0 on
// success or a negative RfError.  Python binds these through ctypes.
#pragma once
#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

typedef void* rf_stream_t;  // cudaStream_t

enum RfError {
  RF_OK = 0,
  RF_ERR_BAD_ARG = -1,
  RF_ERR_CUDA = -2,
  RF_ERR_UNSUPPORTED = -3,
  RF_ERR_NO_MEMORY = -4,
  RF_ERR_STATE = -5,
};

const char* rf_last_error(void);
int rf_version(void);
uint64_t rf_launch_count(void);  // kernels enqueued by this library so far

// ---------------------------------------------------------------- GEMM ----
// out[M,N] = epilogue( x[M,K] . w[N,K]^T ), all row-major, 16-bit in, fp32 acc.
typedef struct RfGemm {
  const void* x; int64_t ldx;
  const void* w; int64_t ldw;
  void* out; int64_t ldo;
  const void* residual; int64_t ldr;  // optional, added last
  const void* bias;                   // optional [N] (dual: [dual_offset+N])
  const void* scale;                  // optional per-output-channel scale [N], same dtype
  const float* row_scale;             // optional per-token fp32 scale [M]
  int32_t M, N, K;
  int32_t dtype;        // 0 fp16, 1 bf16
  int32_t act;          // rf::Act
  int32_t dual_offset;  // >0: second weight block starts dual_offset rows below the first
  int32_t w_int8;       // 1: w is int8 [N,K] (scale required)
  float* ws; uint64_t ws_bytes;  // split-K scratch (fp32 partials), optional
  uint32_t* sem; int32_t sem_count;  // split-K tile semaphores, zero-initialised once
  int32_t* status;      // device status block, optional
  // fused all-reduce over peer memory (world > 1): partial tiles are pushed
  // into every rank's receive buffer, summed in rank order, residual added.
  int32_t ar_world, ar_rank;
  void* const* ar_recv;        // device array [world] of receive-buffer bases
  uint32_t* const* ar_flags;   // device array [world] of flag-array bases
  uint32_t* ar_state;          // local: [0] call counter, [1] finished-CTA counter
  uint64_t ar_recv_bytes;      // bytes of one half of the (double-buffered) receive buffer
  int32_t ar_flag_count;       // flags available per rank
  int32_t force_splits;        // 0 = heuristic
  int32_t force_swap;          // -1 = heuristic, 0/1 forced
  int32_t force_bn;            // 0 = heuristic
  // 1: w is in the tile-major layout (see rf_pack_weight_bytes): block (row tile rt, k block kb) of
  // 128 rows x 64 columns is contiguous, 16-bit blocks already in the 128-byte-swizzled shared-memory
  // image, so one 16 KB (int8: 8 KB) bulk copy per block streams HBM pages front to back.  Rows are
  // padded to 128 per section (dual: gate section, then up section), K to 64; ldw is ignored.
  int32_t w_packed;
  // W8A16 with more than 256 tokens: device scratch for the widened (16-bit, tile-major) weight image, twice
  // the bytes of the int8 image.  Null: the int8 tile is widened inside the main loop for every token count.
  void* w_scratch;
  uint64_t w_scratch_bytes;
  // Tensor parallel, at most 256 tokens: 1 = "publish and exit".  The epilogue only pushes this rank's partial
  // rows (16-byte vectors) into every rank's receive buffer and bumps counter ar_cnt_base + ar_rank on every rank;
  // it does not wait, reduce, add the residual or write `out`.  rf_ar_consume() finishes the all-reduce.
  int32_t ar_publish;
  int32_t ar_cnt_base;         // first of `world` arrival counters in every rank's flag array
  // Optional hint (weight-streaming shapes of at most 256 tokens): device memory the NEXT kernel on the stream will
  // read - normally the next linear layer's weights.  Once a CTA has issued its own last weight load it asks for its
  // share of the first prefetch_bytes of that memory to be brought into L2, so HBM keeps streaming through this
  // kernel's epilogue, the launch gap and the next kernel's prologue.  Never dereferenced; 16-byte aligned.
  const void* prefetch;
  uint64_t prefetch_bytes;
  // 4: `w` is the tile-major int4 image made by rf_pack_w4 / ops.kernels.pack_weight_int4 (w_int8 = 1, w_packed = 1):
  // block (row tile, k block) = 128 rows x 64 columns as 4096 bytes of nibbles (two's complement; inside each group of
  // eight columns the nibbles sit in the order 0,2,4,6,1,3,5,7) followed by the block's scales in the activation dtype,
  // 128 x (64 / min(w_group, 64)) of them.  w_group = 0: no scales in the image, `scale` holds one per output channel.
  int32_t w_bits;
  int32_t w_group;     // 0, 16 (fp4 only), 32, 64 or 128 columns per scale
  // 0: the nibbles are two's-complement integers (W4A16); 1: e2m1 floating-point codes (bit 3 sign, bits 0..2 index into
  // {0, 0.5, 1, 1.5, 2, 3, 4, 6}) as in NVFP4, whose e4m3 block scale times the tensor scale is stored per 16 columns
  // in the image, already multiplied out in the activation dtype.
  int32_t w_fp4;
  // RMSNorm folded around the GEMMs (at most 256 tokens, weights streamed with tokens on the MMA N axis):
  //  * ss_out: this GEMM also writes, for every token and every 128-wide tile of its output columns, the sum of
  //    squares of the finished (residual added, rounded) values: ss_out[tile * ss_ld + token], fp32.  Plain stores in
  //    a fixed layout, so the later sum has a fixed order.
  //  * ss_in: the input rows are un-normalised; the result is scaled per token by
  //    rsqrt(sum_{t < ss_tiles} ss_in[t * ss_ld + token] / ss_dim + ss_eps), which together with norm weights
  //    multiplied into the weight columns beforehand is the RMSNorm that would otherwise run as its own kernel.
  int32_t ss_tiles;
  float* ss_out;
  const float* ss_in;
  int32_t ss_ld, ss_dim;
  float ss_eps;
  int32_t streaming_only;      // 1: never the latency-bound mma.sync kernel (gemm_small.cu), whatever the shape
  // Gate by token (shapes for which rf_gemm_takes_mul returns 1): the activated result of row m, column n is multiplied by
  // mul[mul_row[m] * mul_ld + n] (same dtype), a slice of an embedding table.
  const void* mul; const int32_t* mul_row; int64_t mul_ld;
  float act_limit, act_alpha;  // constants of the activations that have some (rf::ActArgs)
} RfGemm;
// bytes of the tile-major image of a [rows, K] weight with `sections` equal row sections
uint64_t rf_pack_weight_bytes(int64_t rows, int64_t K, int32_t sections, int32_t elem_bytes);
// bytes of the tile-major int4 image (see RfGemm.w_bits) and of one of its blocks
uint64_t rf_pack_w4_bytes(int64_t rows, int64_t K, int32_t sections, int32_t group);
int32_t rf_w4_block_bytes(int32_t group);

int rf_gemm(const RfGemm* g, rf_stream_t stream);
int rf_gemm_takes_mul(const RfGemm* g);   // host-only: can this GEMM apply RfGemm.mul in its epilogue?
// Launch plan of a shape without launching: out[10] = {swap, bn, splits, stages, grid_x, grid_y, smem bytes, k_blocks,
// persistent kernel, two-shot all-reduce}.  Host-only.
int rf_gemm_plan_info(const RfGemm* g, int32_t* out);
// Scratch a split-K launch of this shape would need (bytes of ws, number of sems).
int rf_gemm_scratch(const RfGemm* g, uint64_t* ws_bytes, int32_t* sem_count);
// Same contract with int8 weights [N,K] and a per-output-channel scale (W8A16):
// the int8 tile is widened to the activation dtype inside the mainloop.
int rf_gemm_w8a16(const RfGemm* g, rf_stream_t stream);
// int4 weights (w_bits = 4) with per-channel or group-wise scales: nibbles are widened, and group scales applied, by the
// converter warps of the same main loop.
int rf_gemm_w4a16(const RfGemm* g, rf_stream_t stream);
// CUDA-core skinny GEMM (M <= 8): reference path and small-batch decode.
int rf_gemv(const RfGemm* g, rf_stream_t stream);
// CTAs of the launch rf_gemm / rf_gemm_w8a16 would make for this shape (each bumps the arrival counters once when
// ar_publish is set); negative RfError on a bad shape.  Host-only.
int rf_gemm_grid_ctas(const RfGemm* g);

// Second half of the tensor-parallel all-reduce of a row-parallel GEMM launched with ar_publish: waits (bounded)
// until every rank's arrival counter shows that all `pub_ctas` CTAs of its GEMM have published, sums the ranks'
// partial rows in rank order in fp32, adds the residual, writes `out`, and optionally applies the RMSNorm that
// follows in the layer (norm_mode 1: w * norm(x), 2: (1 + w) * norm(x)) into norm_out.  out may alias residual.
// Partials are fp32 up to RF_AR_F32_MAX_ROWS rows and the activation dtype above.
#define RF_AR_F32_MAX_ROWS 16
typedef struct RfArConsume {
  int32_t M, N;                // rows (tokens) and columns (hidden size); N a multiple of 8
  int32_t world, rank;
  void* const* ar_recv;        // device array [world] of receive-buffer bases (only [rank] is read here)
  uint32_t* const* ar_flags;   // device array [world] of flag-array bases (only [rank] is read here)
  uint32_t* ar_state;          // local state words: [0] call counter, [4] counter value consumed so far, [5] finished CTAs
  uint64_t ar_recv_bytes;      // bytes of one half of the double-buffered receive buffer
  int32_t ar_cnt_base;
  int32_t pub_ctas;            // rf_gemm_grid_ctas() of the producing GEMM
  const void* residual; int64_t ldr;   // optional
  void* out; int64_t ldo;
  const void* norm_w; void* norm_out; int64_t ldn;   // optional fused RMSNorm of the finished rows
  float eps; int32_t norm_mode;
  int32_t* status; int32_t dtype;
} RfArConsume;
int rf_ar_consume(const RfArConsume* a, rf_stream_t stream);

// Two-shot all-reduce for large token counts (prefill), over buffers that every rank allocated at the same offsets
// of its peer-mapped communication region ("symmetric" buffers; the tables hold one base pointer per rank).
// Every rank's row-parallel GEMM has written its partial result [M, N] into its own `partial` buffer.  Rank r owns
// rows [r * ceil(M / world), ...): it reads those rows of EVERY rank's partial over NVLink (reduce-scatter by peer
// loads, summed in rank order in fp32), adds the residual, and writes the finished rows -- and, when norm_mode != 0,
// the RMSNorm of them -- into every rank's `out` (and `norm_out`) buffer (all-gather by peer stores).  The residual is
// read from this rank's own `out` buffer when add_residual is set (the residual stream lives there).  With out_local
// the finished rows are written on their owner only: each rank then holds M / world rows of the residual stream, and
// what crosses NVLink is a reduce-scatter of the partials plus an all-gather of the normalised rows.  Flags:
// world "partial ready" + world "rows written" words per rank at flag_base; state word 6 is the epoch.
typedef struct RfArRows {
  int32_t M, N, world, rank;
  void* const* partial_tab;    // device array [world]: every rank's partial [M, N]
  void* const* out_tab;        // device array [world]: every rank's destination [M, N]
  void* const* norm_tab;       // device array [world]: every rank's normalised destination (optional)
  uint32_t* const* ar_flags;   // device array [world] of flag-array bases
  uint32_t* ar_state;
  int32_t flag_base;
  int32_t add_residual;
  const void* norm_w; float eps; int32_t norm_mode;
  int32_t* status; int32_t dtype;
  int32_t out_local;           // 1: the finished rows stay on their owner (sequence-sharded residual stream); only the
                               // normalised rows are gathered on every rank
} RfArRows;
int rf_ar_rows(const RfArRows* a, rf_stream_t stream);


// ------------------------------------------------------ norms / glue ----
int rf_rmsnorm(const void* x, const void* residual, const void* w, void* y, void* residual_out,
               const void* mod, int rows_per_mod, int rows, int H, int64_t ldx, int64_t ldy,
               float eps, int mode, int dtype, rf_stream_t stream);
int rf_layernorm(const void* x, const void* w, const void* b, void* y, int rows, int H,
                 int64_t ldx, int64_t ldy, float eps, int dtype, rf_stream_t stream);
int rf_l2norm(const void* x, void* y, int rows, int H, float eps, float out_scale, int dtype,
              rf_stream_t stream);
int rf_gated_residual(void* x, const void* y, const void* mod, int rows_per_mod, int rows, int H,
                      int dtype, rf_stream_t stream);

// Per-head RMSNorm(q,k) -> RoPE -> KV page insert on a packed [tokens, (Hq+2Hkv)*hd] buffer.
typedef struct RfRopeKv {
  void* qkv; int64_t ld;
  void* q_out; int64_t ldq;        // optional: rotated q goes here instead of in place
  int32_t tokens, Hq, Hkv, hd, rot_dim;
  const void* q_norm_w; const void* k_norm_w;  // optional [hd]
  float eps; int32_t norm_mode;     // bit0: (1+w) weight
  const float* cos; const float* sin;  // [max_pos, rot_dim/2] fp32, optional
  const int32_t* pos; int32_t pos_stride;  // [tokens, pos_stride]
  const int8_t* axis_of_freq;       // optional [rot_dim/2]: which position axis a frequency uses
  void* k_pool; void* v_pool;       // optional [pages, Hkv, 16, hd]
  const int32_t* page_table; int32_t pt_stride;  // [seqs, pt_stride]
  const int32_t* seq_of_tok;        // optional [tokens]; default token index
  const int32_t* cache_pos;         // optional [tokens]; default pos[tok, 0]
  int32_t rope_before_norm;
  int32_t write_k_inplace;          // also write rotated k back into qkv
  int32_t dtype;
  int32_t v_norm;                   // unweighted RMSNorm of every value head (in place, before the cache insert)
} RfRopeKv;
int rf_qk_norm_rope_kv(const RfRopeKv* a, rf_stream_t stream);

// out[i] = table[ids[i]] (row gather); ids < 0 give zero rows.  scale multiplies (Gemma sqrt(H)).
int rf_embedding(const void* table, const int32_t* ids, void* out, int n_ids, int H, int64_t ldo,
                 float scale, int dtype, const void* row_scale_i8, rf_stream_t stream);
// dst[rows[i]] = src[i]  (splice vision rows into text rows)
int rf_scatter_rows(void* dst, const void* src, const int32_t* rows, int n, int H, int64_t ldd,
                    int64_t lds, int accumulate, int dtype, rf_stream_t stream);
// Elementwise: op 0 add, 1 mul, 2 silu(a)*b, 3 gelu_tanh(a)*b, 4 a + alpha*b, 5 gelu_tanh(a),
// 6 gelu_erf(a), 7 silu(a), 8 a*alpha, 9 sigmoid(a)*b, 10 a*(broadcast row vector b), 11 tanh(a)
int rf_eltwise(int op, const void* a, const void* b, void* out, int64_t n, int64_t b_period,
               float alpha, int dtype, rf_stream_t stream);
int rf_cast_u8_f16(const uint8_t* src, void* dst, int64_t n, float scale, float shift, int dtype,
                   rf_stream_t stream);
// Greedy top-1 over the last dim; two-stage, writes int32 ids (and fp32 max when vals != null).
// offset is added to every id (vocab shard base).
int rf_argmax(const void* logits, int rows, int V, int64_t ld, int32_t* out_ids, float* out_vals,
              int32_t offset, void* scratch, uint64_t scratch_bytes, int dtype, rf_stream_t stream);
uint64_t rf_argmax_scratch_bytes(int rows, int V);


// ----------------------------------------------------------- attention ----
// q/out: [q_rows_total, Hq*hd] (pitch ldq/ldo).  KV comes either from the paged
// pool ([pages, Hkv, 16, hd], page_table[seq, i] -> page id) or from contiguous
// rows k/v[kv_rows_total, Hkv*hd].  The pool must only ever hold finite values
// (it is zero-filled at creation): masked tokens still pass through the MMA.
typedef struct RfAttn {
  const void* q; int64_t ldq;
  void* out; int64_t ldo;
  int64_t q_rows_total;
  const void* k_pool; const void* v_pool; int64_t pool_pages;
  const int32_t* page_table; int32_t pt_stride;
  const void* k; const void* v; int64_t ldk, ldv; int64_t kv_rows_total;
  int32_t num_seqs, Hq, Hkv, hd;
  const int32_t* q_start;   // [num_seqs] first q row (prefill)
  const int32_t* q_len;     // [num_seqs] (prefill)
  const int32_t* kv_start;  // [num_seqs] first kv row (contiguous mode)
  const int32_t* kv_len;    // [num_seqs] valid kv tokens, device
  int32_t max_q_len, max_kv_len;  // host-side bounds used for grid sizing
  int32_t causal;           // q row i sits at position kv_len - q_len + i
  int32_t window;           // > 0: sliding window
  const uint8_t* mask; int64_t mask_ld, mask_seq_stride;  // optional boolean [q, kv] per sequence
  const int32_t* seg_q; const int32_t* seg_k;             // optional segment ids per q row / kv row
  float scale;              // <= 0: 1/sqrt(hd)
  float* ws; uint64_t ws_bytes;  // decode split-KV scratch, optional
  int32_t* status; int32_t dtype;
  // Options of the paged forms:
  const int32_t* slot;      // page-table row of every sequence (null: the sequence's own index)
  int32_t chunk;            // > 0: position i sees j only if i / chunk == j / chunk (positions count from the sequence's start)
  const float* sink;        // [Hq]: the softmax denominator also holds exp(sink[h])
  const void* gate; int64_t ld_gate;   // [rows, Hq * hd]: the result is multiplied by sigmoid(gate) before it is rounded
  int32_t gate_by_head;     // 1: gate is [rows, Hq], one number per head
  int32_t keep_first;       // with a window: the first keep_first positions of the sequence stay visible
  const float* slopes;      // [Hq]: slopes[h] * (i - j) is taken off the scores of position i (paged forms)
  const float* rates;       // [Hq], with slopes: slopes[h] * ln(1 + rates[h] * (i - j)) instead
  // rf_attn_decode by row: with `pos`, query row r is position pos[r] of sequence seq_of_row[r] (null: r) and sees what its
  // chunk or window leaves of everything up to itself; kv_len is not used and num_seqs counts rows.
  const int32_t* seq_of_row; const int32_t* pos;
  int32_t vd;               // size of a value head (0: hd); contiguous rows with hd = 192 take 128, out is [rows, Hq * vd]
} RfAttn;
int rf_attn_prefill(const RfAttn* a, rf_stream_t stream);
int rf_attn_decode(const RfAttn* a, rf_stream_t stream);
uint64_t rf_attn_decode_scratch_bytes(int num_seqs, int Hq, int hd);
// The most scratch rf_attn_decode asks for at any number of sequences and keys.
uint64_t rf_attn_decode_scratch_bound(int Hq, int Hkv, int hd);


// --------------------------------------------- linear attention (GDN) ----
// Causal depthwise conv1d (kernel size 4) + optional SiLU over C channels of packed varlen rows,
// with a carried state [slots, K-1, C] (oldest row first) that is read, then replaced by the last
// K-1 inputs of every sequence.  q_start/q_len null: one token per sequence (decode), row = seq.
// x and y must not alias.
typedef struct RfConv1d {
  const void* x; int64_t ldx;
  void* y; int64_t ldy;
  const void* w;            // [C, K]
  void* state;              // [slots, K-1, C]
  const int32_t* q_start; const int32_t* q_len; const int32_t* slot;   // device, [num_seqs]; slot null: seq
  int32_t num_seqs, max_q_len, C, K, silu, dtype;
} RfConv1d;
int rf_causal_conv1d(const RfConv1d* a, rf_stream_t stream);

// Gated delta rule over n tokens per sequence (n = 1: decode step):
//   beta = sigmoid(b), g = -exp(A_log) * softplus(a + dt_bias), q,k L2-normalised, q /= sqrt(Dk)
//   S *= exp(g);  kv = k^T S;  d = (v - kv) * beta;  S += k (x) d;  o = q^T S
// qkv rows hold [q: Hk*Dk | k: Hk*Dk | v: Hv*Dv]; value head h reads key head h / (Hv/Hk).
// state: fp32 [slots, Hv, Dk, Dv]; fresh[seq] != 0 starts that sequence from a zero state.
typedef struct RfGdn {
  const void* qkv; int64_t ld;
  const void* b; const void* a; int64_t ld_ba;     // [rows, >= Hv] each
  void* out; int64_t ldo;                           // [rows, Hv*Dv]
  float* state;
  const float* A_log; const float* dt_bias;         // [Hv] fp32
  const int32_t* q_start; const int32_t* q_len; const int32_t* slot; const int32_t* fresh;
  int32_t num_seqs, Hk, Hv, Dk, Dv, dtype;
} RfGdn;
int rf_gdn_recurrent(const RfGdn* a, rf_stream_t stream);
// Same contract, evaluated 64 tokens at a time on the tensor cores (prefill; decode keeps the recurrent kernel).
int rf_gdn_chunked(const RfGdn* a, rf_stream_t stream);
// y[t, h, :] = (w * rmsnorm(x[t, h, :])) * silu(z[t, h, :]), D values per (token, head)
int rf_rmsnorm_gated(const void* x, int64_t ldx, const void* z, int64_t ldz, const void* w, void* y, int64_t ldy,
                     int tokens, int heads, int D, float eps, int dtype, rf_stream_t stream);
// a[t, c] *= sigmoid(g[t, c]) (output gate of the gated full-attention layers)
int rf_sigmoid_gate(void* a, int64_t lda, const void* g, int64_t ldg, int rows, int cols, int dtype, rf_stream_t stream);
// helpers of the chunked delta-rule formulation
int rf_cumsum_f32(const float* x, float* y, int rows, int n, rf_stream_t stream);
int rf_unit_tril_inv_f32(const float* m, float* out, int batch, int n, rf_stream_t stream);


// ----------------------------------- decoders with per-layer mixers ----
// Where the rows of a launch belong: row r is one token of sequence seq_of_row[r] (null: row = sequence, one token each),
// sequence s occupies rows [q_start[s], q_start[s] + q_len[s]) (null: one row), keeps its recurrent state and its page-table
// row in slot[s] (null: s), and pos[r] is the row's position in its sequence.  A sequence whose first row has position 0
// starts from an empty state.
typedef struct RfRows {
  const int32_t* seq_of_row; const int32_t* q_start; const int32_t* q_len; const int32_t* slot; const int32_t* pos;
  const int32_t* page_table; int32_t pt_stride; int32_t num_seqs;
} RfRows;

// The fp32 residual stream between two sublayers, one launch:
//   v = x[row]  (or the embedding row table[ids[row]] when x is null)
//   v += y[row]  or, with y_norm_w,  v += y / rms(y) * y_norm_w          (the sublayer output that is still outstanding)
//   x_out = v (fp32), x_cast = v (activation dtype)
//   h = v / rms(v) * norm_w;  with `shift`: out = h + (h_prev - h) * shift, h_prev the h of the sequence's previous token
//   (carried over launches in shift_state[slot], zeros before the first token); without: out = h.
// Embedding rows are multiplied by embed_scale (0 counts as 1); with table2 the row of the token pair (previous token, token) is
// added to them: (previous * mul_prev + token * mul_cur) mod buckets, row `buckets` for a sequence's first token; last_token [slots]
// carries every sequence's last token (not together with `shift`).  The outstanding output is multiplied by y_mult (0 counts as 1)
// when it is added.  With y_picks > 0 the outstanding output is the sum of y_picks rows of y, those
// that y_slots[row * y_picks ...] names (negative: none): the experts' results of a mixture of experts.
// y_self_w [rows] adds y_self_w[row] * y_self[row] to that sum (experts whose output is their input).
// With conv_w (decode rows only: every row is a sequence of its own) the normalised row, rounded to the activation dtype, goes through
// the input convolution before it is written: out = h + sum_k conv_w[k] h[t - (taps - 1) + k], the last taps - 1 rows h carried in
// conv_state [slots, taps - 1, H], oldest first (portions: rf_conv_silu with `add` behind this step, same state).
// H is the (padded, multiple of 8) row length, dim the true one that the means run over.  x_out must not alias x when
// `shift` is set.  row_idx (optional) selects the rows that are processed (not together with shift).
typedef struct RfStreamNorm {
  const float* x; const void* table; const int32_t* ids; const int32_t* row_idx;
  const void* y; const float* y_norm_w;
  float* x_out; void* x_cast;
  const float* norm_w; void* out;
  const float* shift; float* shift_state;
  RfRows rows;
  int32_t n_rows, H, dim; float eps; int32_t dtype;    // dtype 2: fp32 activations
  float embed_scale;
  const int32_t* y_slots; int32_t y_picks;
  float y_mult;
  const void* table2; int32_t* last_token; int64_t mul_prev, mul_cur; int32_t buckets;
  const void* y_self; const float* y_self_w;
  const float* conv_w; void* conv_state; int32_t conv_taps;
} RfStreamNorm;
int rf_stream_norm(const RfStreamNorm* a, rf_stream_t stream);

// out[M, N] = act(x[M, K] . w[N, K]^T) in true fp32 (row-major operands, no tensor cores): the linear layers of a model that
// is served in 32 bits.  Uses x, w, out, their pitches, M, N, K, row_scale, dual_offset and act (with its constants) of RfGemm.
int rf_gemm_f32(const RfGemm* g, rf_stream_t stream);

// g[r, c] *= table[ids[r] * ld_table + col0 + c] for c < cols (a gate multiplied by a per-token embedding slice)
int rf_token_gate(void* g, int64_t ldg, const void* table, int64_t ld_table, const int32_t* ids, int32_t col0, int32_t rows,
                  int32_t cols, int32_t dtype, rf_stream_t stream);

// Per-head linear map y[r, h, n] = sum_k x[r, h, k] w[h, n, k]; head h of row r starts at x + r * ldx + h * xs
// (y + r * ldy + h * ys).  Sizes n, k, xs, ys and pitches are multiples of 8.
typedef struct RfHeadLinear {
  const void* x; int64_t ldx; int32_t xs;
  void* y; int64_t ldy; int32_t ys;
  const void* w;
  int32_t rows, heads, n, k, dtype;
} RfHeadLinear;
int rf_head_linear(const RfHeadLinear* a, rf_stream_t stream);

// Latent-attention cache: one row of `rank` (padded to a multiple of 16) values per token, pool [pages, 16, rank], or, with a
// rotated key part that all heads share, [pages, 16, rank + rot_pad] (rot values behind the latent, padded to a multiple of 16).
// rf_latent_insert: c = x / rms(x) * norm_w (mean over the true rank), stored at the row's position; x holds the rotated part at
// column `rank`, turned by the row's position on the way (RfHeadRotate).  With q also the rows' query latents (their own norm, in
// place).  x null: the query latents alone (a layer that attends over another layer's cache).
typedef struct RfLatentInsert {
  const void* x; int64_t ldx; const float* norm_w; void* pool; RfRows rows;
  int32_t n_rows, rank, rank_true; float eps;
  int32_t rot, rot_pad; const float* cos; const float* sin;
  void* q; int64_t ldq; const float* q_norm; int32_t q_rank, q_rank_true;
} RfLatentInsert;
int rf_latent_insert(const RfLatentInsert* c, int32_t dtype, rf_stream_t stream);
// Rotation of `dims` values of every head in neighbouring pairs: (u, v) of pair i at position p becomes (u c - v s, v c + u s) with
// c, s = cos / sin[p, i] (tables [positions, dims / 2]).  Head h of row r starts at x + r * ldx + h * xs (to y likewise, possibly in
// place); values from dims to dims_pad (a multiple of 8) are written as zeros.
typedef struct RfHeadRotate {
  const void* x; int64_t ldx; int32_t xs;
  void* y; int64_t ldy; int32_t ys;
  const int32_t* pos; const float* cos; const float* sin;
  int32_t rows, heads, dims, dims_pad;
} RfHeadRotate;
int rf_head_rotate(const RfHeadRotate* a, int32_t dtype, rf_stream_t stream);
// The per-head map of the queries into the latent space together with the insertion and / or the rotation above (either may be
// null; one launch in 16 bits): what a decode step does between the query projection and the attention.
int rf_latent_absorb(const RfHeadLinear* q, const RfLatentInsert* c, const RfHeadRotate* t, rf_stream_t stream);
// Dense copies of the latents that sequences can see: the last kv_len[s] cached rows of sequence s, its own new rows (already
// inserted) included, to rows [kv_start[s], kv_start[s] + kv_len[s]) of out.  max_len: host bound of kv_len.
int rf_latent_gather(const void* pool, void* out, const RfRows* rows, const int32_t* kv_start, const int32_t* kv_len, int32_t rank,
                     int32_t max_len, int32_t dtype, rf_stream_t stream);

// Attention in the latent space (keys and values folded into the queries and the output): every row attends from its own
// position to the window before it, score = (q[r, h] . c[j]) * scale, o[r, h] = sum_j softmax(score)_j c[j].
// q, o: [rows, heads, rank] dense.  window <= 0: no lower bound.  max_kv: host bound of the keys one row sees.
// With vrank > 0 only the first vrank of the rank cached columns are values (the others are a rotated key part): o is [rows, heads, vrank].
typedef struct RfLatentAttn {
  const void* q; void* o; const void* pool;
  RfRows rows;
  int32_t n_rows, heads, rank, window, max_kv; float scale; int32_t dtype;
  float* ws; uint64_t ws_bytes;      // split partials, optional
  int32_t vrank;
} RfLatentAttn;
int rf_latent_attn(const RfLatentAttn* a, rf_stream_t stream);
uint64_t rf_latent_attn_scratch_bytes(int rows, int heads, int rank, int max_kv);

// Grouped-head attention over paged K/V pools [pages, kv_heads, 16, hd]: what lies between the input projection and the
// attention, in one launch and in fp32 - RMSNorm of every query and key head over its true size `dim` (optional), rotation of the
// first rot_dims dimensions (rotate-half pairs, cos / sin [positions, rot_dims / 2]), value mixing, insertion of keys and values
// at the row's position.  A row holds heads * hd query values, then kv_heads * hd keys at k_off and values at v_off, every head
// padded with zeros to hd; queries are replaced in place.
// Value mixing: the first mixing layer stores its values in v_first [rows, kv_heads, vdim], later ones take
// v = (1 - v_lambda) v + v_lambda v_first.
enum RfVMix { RF_VMIX_NONE = 0, RF_VMIX_FIRST = 1, RF_VMIX_MIX = 2 };
typedef struct RfQkvInsert {
  void* qkv; int64_t ld; int32_t k_off, v_off;
  const float* q_norm; const float* k_norm; const float* cos; const float* sin;
  void* v_first; void* k_pool; void* v_pool;
  RfRows rows;
  int32_t n_rows, heads, kv_heads, hd, dim, vdim, rot_dims, v_role; float v_lambda, eps; int32_t dtype;
  int32_t norm_all;                    // 1: one RMSNorm over all query heads of a row and one over all key heads; q_norm [heads, hd],
                                       // k_norm [kv_heads, hd] (per-head norms: [hd])
  // Causal convolution per channel of queries, keys and values ahead of the norms: y[t] = sum_k w[k] x[t - (taps - 1) + k].  The last
  // taps - 1 rows of [queries | keys | values] are carried in conv_state [slots, taps - 1, (heads + 2 kv_heads) * hd], oldest first.
  // conv_w: [taps, (heads + 2 kv_heads) * hd].  The rows are read only, queries go to q_out [n_rows, heads * hd].
  const float* conv_w; void* conv_state; void* q_out; int32_t taps, max_q_len;
  float growth; int32_t growth_every;  // every > 0: queries of position p times 1 + growth * ln(floor((p + 1) / every) + 1)
} RfQkvInsert;
int rf_qkv_insert(const RfQkvInsert* a, rf_stream_t stream);
// Attention by row on the CUDA cores in fp32, any head size up to 2048 and any scale: the by-row form of rf_attn_decode (pos,
// seq_of_row, slot, chunk, window, sink, gate, slopes) for 32-bit models and heads the tensor-core kernels do not take.
int rf_attn_rows(const RfAttn* a, rf_stream_t stream);

// Causal convolution per channel over packed rows, silu applied: y[t] = silu(bias + sum_k w[k] x[t - (taps - 1) + k]).  The last
// taps - 1 inputs of every sequence are carried in state [slots, taps - 1, channels], oldest first.  w: [taps, channels] fp32.
// `add`: y[t] = x[t] + the sum, without silu.  `ring`: state is [slots, taps, channels], the input of position p in row p mod taps.
typedef struct RfConvSilu {
  const void* x; int64_t ldx; void* y; int64_t ldy;
  const float* w; const float* bias; void* state;
  RfRows rows;
  int32_t max_q_len, channels, taps, dtype;
  int32_t add, ring;
} RfConvSilu;
int rf_conv_silu(const RfConvSilu* a, rf_stream_t stream);

// Selective scan (Mamba): with dt = softplus(step size + dt_bias),  S = 2^(dt a2) S + dt x B,  y = (S C + d x) silu(z).
// a2 [inner, states] is -exp(A_log) / ln 2; rows of bc hold [step-size input: rank | B: states | C: states]; state: fp32
// [slots, inner, states].  Padding states have a2 = 0 and zero B and C.
// The recurrent form computes the step sizes itself from w_dt [inner, rank] (row-major, activation dtype) and takes any portions;
// the scan form takes them projected (dt [rows, inner], before the bias) and is for prefill-sized portions.
typedef struct RfMamba1 {
  const void* x; int64_t ldx; const void* z; int64_t ldz; const void* bc; int64_t ld_bc; const void* dt; int64_t ld_dt;
  const void* w_dt; const float* dt_bias; const float* a2; const float* d;
  float* state; void* out; int64_t ldo;
  RfRows rows;
  int32_t inner, states, rank, dtype;
} RfMamba1;
int rf_mamba1_recurrent(const RfMamba1* a, rf_stream_t stream);
int rf_mamba1_scan(const RfMamba1* a, rf_stream_t stream);

// Gated delta rule with an output norm and gate (see kernels/delta_rule.cu).  Rows of x hold [q: kv_heads * dim | k: kv_heads * dim |
// v: heads * vdim] behind the short convolution and silu; head h uses query / key head h / (heads / kv_heads).  rate [heads] = exp(A_log);
// state fp32 [slots, heads, dim, vdim]; padding dimensions of q, k and v are zero.  b, a: [rows, >= heads]; gate [rows, heads * vdim].
// With conv_w (decode steps of the recurrent form) x are the projections: conv_w [taps, channels] and the ring of rf_conv_silu.
typedef struct RfDelta {
  const void* x; int64_t ldx; const void* b; const void* a; int64_t ld_ba; const void* gate; int64_t ldg;
  const float* rate; const float* dt_bias; const float* norm_w;
  float* state; void* out; int64_t ldo;
  RfRows rows;
  int32_t heads, kv_heads, dim, dim_true, vdim, vdim_true; float eps; int32_t dtype;
  const float* conv_w; void* conv_state; int32_t taps;
} RfDelta;
int rf_delta_recurrent(const RfDelta* a, rf_stream_t stream);
// Same contract, 64 tokens at a time (prefill-sized portions; 16-bit activations, dim 64 / 128, vdim a multiple of 32).  The
// sequences' rows are [row0, row0 + rows).
int rf_delta_chunked(const RfDelta* a, int row0, int rows, rf_stream_t stream);
int rf_delta_chunked_supported(int dim, int vdim, int dtype);

// HGRN2 linear attention (what a gate takes from the state it gives to the new value), over packed input rows [q | f | v]:
//   q = silu(q), f = lower + (1 - lower) * sigmoid(f + f_bias), S = diag(f) S + (1 - f) v^T, o = S^T q,
//   out = o / rms(o) * norm_w per head (mean over the true value size; null norm_w: plain o)
// state: fp32 [slots, heads, dim, vdim].  Padding channels of dim have lower = 1, padding value columns are zero.
typedef struct RfHgrn2 {
  const void* x; int64_t ldx; int32_t f_off, v_off;
  const float* f_bias; const float* lower; const float* norm_w;
  float* state; void* out; int64_t ldo;
  RfRows rows;
  int32_t heads, dim, vdim, vdim_true; float eps; int32_t dtype;
  int32_t* status;                     // device status block, optional
} RfHgrn2;
int rf_hgrn2_recurrent(const RfHgrn2* a, rf_stream_t stream);
// Same contract, evaluated block by block (prefill-sized portions; 16-bit activations).
int rf_hgrn2_chunked(const RfHgrn2* a, rf_stream_t stream);
int rf_hgrn2_chunked_supported(int dim, int vdim, int dtype);


// ------------------------------------------------- mixture of experts ----
// Router: scores = sigmoid(logits) (score_fn 0) or softmax(logits) (1); the k experts with the largest
// (score + bias) are selected, ties to the lower index; weights are the UNBIASED scores, divided by their
// sum when norm_topk, times scale.  Any of out_ids [rows,k], out_w [rows,k], dense_w [rows,E] (zero for
// unselected experts) may be null.  E <= 256, k <= 32.
int rf_moe_select(const void* logits, int64_t ld, const float* bias, int rows, int E, int k, int score_fn,
                  int norm_topk, float scale, int32_t* out_ids, float* out_w, void* dense_w, int64_t ldd, int dtype,
                  rf_stream_t stream);
// h[t, e*I + c] *= dense_w[t, e] for the E routed expert blocks of width I (dense-einsum expert MLP)
int rf_moe_scale_blocks(void* h, int64_t ldh, const void* dense_w, int64_t ldd, int rows, int E, int I, int dtype,
                        rf_stream_t stream);


// Grouped expert GEMM.  The (token, pick) pairs of a batch are bucketed by expert (rf_moe_group), their rows are
// gathered in that order, and ONE persistent launch multiplies every 128-row block of one expert's rows with that
// expert's weights out of the packed expert bank: out[s, :] = act(x[s, :] . W_e^T) (* row_scale[s]) for every sorted
// row s of expert e.  Only the experts that were picked are read, and only for as many row blocks as they have rows.
//   up / gate projections: the bank stacks the experts along N (rt_per_expert row tiles apart, kb_per_expert = 0);
//   down projection:       the bank concatenates the experts along K (kb_per_expert k blocks apart, rt_per_expert = 0).
typedef struct RfMoeGroupedGemm {
  const void* x; int64_t ldx;          // sorted rows [max_rows, K]
  const void* w;                       // tile-major image of the whole expert bank (rf_pack_weight_bytes layout)
  void* out; int64_t ldo;              // [max_rows, N]
  const float* row_scale;              // optional [max_rows] (routing weight of the row)
  const int32_t* tiles;                // device: [0] number of row blocks, then {expert, first row, end row, 0} per block
  int32_t max_rows, N, K;              // upper bound of sorted rows; per-expert GEMM shape
  int32_t dual, act;                   // dual = 1: GLU pair (gate section, then up section of the bank)
  int32_t bank_section_row_tiles;      // 128-row tiles of one section of the bank image
  int32_t bank_kb_total;               // 64-column k blocks of one row tile of the bank image
  int32_t rt_per_expert, kb_per_expert;
  int32_t dtype; int32_t* status;
  float act_limit, act_alpha;          // rf::ActArgs
} RfMoeGroupedGemm;
int rf_moe_grouped_gemm(const RfMoeGroupedGemm* a, rf_stream_t stream);
// Bucket the picks by expert.  ids / w: [rows, k] (rf_moe_select).  Outputs (device): slot_of [rows*k] = sorted row
// of pick (t, j); token_of_slot [rows*k]; slot_w [rows*k] (fp32 routing weight per sorted row); tiles = the list
// rf_moe_grouped_gemm takes (1 + 4 * (rows*k/128 + E) int32).  One CTA; rows * k <= 1 << 20, E <= 256.
int rf_moe_group(const int32_t* ids, const float* w, int rows, int k, int E, int32_t* slot_of, int32_t* token_of_slot,
                 float* slot_w, int32_t* tiles, rf_stream_t stream);
// out[t, :] += sum_j y[slot_of[t, j], :]  (fp32, picks in order j = 0..k-1, one rounding)
int rf_moe_combine(void* out, int64_t ldo, const void* y, int64_t ldy, const int32_t* slot_of, int rows, int k, int H,
                   int dtype, rf_stream_t stream);


// Router and expert plan, two launches.  logits = x w^T in fp32, scores = softmax (or sigmoid) over all experts, choice scores =
// scores + correction; only experts of the `keep` best of `groups` equal groups (a group counts as much as its best expert) can be
// chosen, the k largest choice scores are; weights are the chosen experts' scores, divided by their sum with norm_topk, times
// scale.  Outputs: ids / weights [rows, k]; rank [rows, k] = the pick's place among its expert's picks; start [experts];
// the tile list (the count in words 0 and 3, entries of four words from word 4 on: tiles + 3 is a list for rf_moe_grouped_gemm;
// blocks of tile_rows rows, with shared_tiles followed by blocks of the shared expert, number `experts`, over sorted rows
// [rows * k, rows * k + rows)).  With `scatter` (few rows) also
// what rf_moe_gather otherwise writes: slot_of [rows, slot_ld] (sorted row of every pick, then of the shared expert),
// token_of_slot and slot_w.  counters: experts + 1 words, zero before the first launch and left zero.
// RF_MOE_CHOSEN: the correction is a bias of the logits; the k largest logits are chosen and the weights are the softmax over the
// chosen ones.  identity: the last this many experts have no weights, their output is their input; picks of them get no row, their
// weights are added up in self_w [rows].  shared_gate: w has one more row behind the experts', sigmoid of its logit is the shared expert's weight (else 1).
enum RfMoeScore { RF_MOE_SIGMOID = 0, RF_MOE_SOFTMAX = 1, RF_MOE_CHOSEN = 2 };
typedef struct RfMoeRouter {
  const void* x; int64_t ldx; const void* w; const float* correction;
  int32_t* ids; float* weights; int32_t* rank; int32_t* counters; int32_t* start; int32_t* tiles;
  int32_t* slot_of; int32_t* token_of_slot; float* slot_w;
  int32_t rows, experts, width, k, groups, keep, score_fn, norm_topk; float scale;
  int32_t tile_rows, slot_ld, has_shared, shared_tiles, scatter, dtype;
  float* logits;                       // scratch, rf_moe_router_scratch_bytes(rows, experts + shared_gate)
  int32_t shared_gate;
  int32_t identity; float* self_w;
} RfMoeRouter;
uint64_t rf_moe_router_scratch_bytes(int rows, int experts);
int rf_moe_router(const RfMoeRouter* a, rf_stream_t stream);
// Copies every row of x to the sorted rows of its picks (and writes slot_of, token_of_slot, slot_w).
int rf_moe_gather(const RfMoeRouter* a, void* out, int64_t ldo, rf_stream_t stream);

// Expert GEMMs of few rows over the tile list of rf_moe_router: out[s] = act(x[row of s] W_e^T) (* slot_w[s]); the row is
// token_of_slot[s], or s itself where that is null.  16-bit: banks are tile-major images as in rf_moe_grouped_gemm, the shared
// expert has its own; tiles of 16 or 32 rows.  32-bit: banks are plain [experts][n][k] matrices (dual: all gates, then all ups);
// tiles of 64 rows.
typedef struct RfMoeExperts {
  const void* x; int64_t ldx; const void* w; const void* w_shared; void* out; int64_t ldo;
  const int32_t* tiles; const int32_t* token_of_slot; const float* slot_w;
  int32_t max_tiles, experts, n, k, shared_n, shared_k, dual, tile_rows;
  int32_t bank_section_row_tiles, bank_kb_total, rt_per_expert, kb_per_expert, shared_section_row_tiles, shared_kb_total, dtype;
  int32_t act;                         // dual: rf::Act of two operands (0 counts as silu(g) u); else of one operand (two-operand ones count as none)
  float act_limit, act_alpha, shared_limit;   // its constants; the shared expert has a limit of its own
} RfMoeExperts;
int rf_moe_experts(const RfMoeExperts* a, rf_stream_t stream);


// ------------------------------------------------------------- KV pool ----
int64_t rf_kvpool_create(int32_t num_pages, int32_t max_seqs, int32_t pages_per_seq);
int rf_kvpool_destroy(int64_t h);
int rf_kvpool_reserve(int64_t h, int32_t seq, int32_t tokens, int32_t* table_row);
int rf_kvpool_release(int64_t h, int32_t seq);
int32_t rf_kvpool_free_pages(int64_t h);


// ------------------------------------------------ peer memory (TP) ----
int rf_comm_alloc(uint64_t bytes, void** out);   // cudaMalloc + zero fill
int rf_comm_free(void* p);
int rf_ipc_export(void* p, uint8_t* handle64);
int rf_ipc_import(const uint8_t* handle64, void** out);
int rf_ipc_close(void* p);
int rf_tp_argmax_merge(void* const* aux, uint32_t* const* flags, int flag_base, uint32_t* state, int world,
                       int rank, int rows, int max_rows, const float* vals, int32_t* ids, int32_t* status,
                       rf_stream_t stream);
int rf_peer_barrier(uint32_t* const* flags, int flag_base, uint32_t* state, int world, int rank,
                    int32_t* status, rf_stream_t stream);

#ifdef __cplusplus
}
#endif
