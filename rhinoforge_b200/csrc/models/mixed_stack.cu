// Executor of decoders with per-layer mixers (see mixed_stack.h).  Host-side C++ only: every device operation is one of the
// kernels in ../kernels, enqueued on the caller's stream.
#include "mixed_stack.h"

#include <algorithm>
#include <memory>
#include <vector>

#include "../common/dtype.cuh"
#include "../common/host_util.h"
#include "../common/status.h"
#include "../runtime/handle_registry.h"

namespace rf {

// Prefill-sized portions under one window: how many keys each sequence sees and how the sequences are grouped so that the
// expanded keys and values of a group fit the buffers.  kv_start / kv_len are uploaded once per forward, ahead of the layer
// loop: the attention kernels read them before their dependency wait, so no kernel of the loop may write them.
struct PortionGroup { int seq0, seqs, total, max_len, max_q; };
struct WindowPlan {
  int window = 0;
  const int32_t* kv_start = nullptr;      // device, one per prefill-sized sequence
  const int32_t* kv_len = nullptr;
  std::vector<PortionGroup> groups;
};

struct MixedStack {
  RfMixedConfig cfg;
  std::vector<RfMixedLayer> layers;
  std::vector<WindowPlan> windows;        // one per distinct window of the expanded layers
  uint8_t* base = nullptr;
  uint64_t off_x[2] = {}, off_h = 0, off_cast = 0, off_wide = 0, off_mix = 0, off_y = 0, off_side = 0, off_qlat = 0, off_olat = 0,
           off_ctx = 0, off_kv = 0, off_kvmeta = 0, off_attn_ws = 0, off_head = 0, off_argmax = 0, off_sk_ws = 0, off_sk_flags = 0,
           off_status = 0, off_vfirst = 0, off_q = 0, off_conv = 0, off_bc = 0, off_dt = 0, off_moe = 0, off_xg = 0, off_hg = 0, off_yg = 0, off_router = 0, off_self = 0, total = 0;
  uint64_t attn_ws_bytes = 0, argmax_bytes = 0, sk_ws_bytes = 0, rows_ws_bytes = 0;
  int moe_tiles = 0;      // tile-list entries of any mixture-of-experts layer
  int lat_rows = 0;       // rows one latent-space attention launch takes
  int ctx_rows = 0;       // rows of expanded keys / values one group of portions takes
  int cur = 0;            // which stream buffer holds the last forward's rows
  // the sublayer output that is still to be added behind the last layer
  struct Pending { const void* y = nullptr; const float* norm = nullptr; const int32_t* slots = nullptr; int picks = 0; const void* self = nullptr; const float* self_w = nullptr; } tail;
  const int32_t* full_len = nullptr;      // device: cached tokens, new ones included, of every prefill-sized sequence
  int max_full = 0, max_long_q = 0;
  bool planned = false;
  static constexpr int kSkFlags = 1024;
  static constexpr int kMoeExperts = 260;     // 256 experts and a ticket, in whole int4
  static constexpr int kMoeSmallRows = 256;   // up to here the experts' weights are streamed past the rows

  size_t esz() const { return cfg.dtype == kF32 ? 4 : 2; }
  bool fp32() const { return cfg.dtype == kF32; }
  template <typename P = void> P* at(uint64_t off) const { return reinterpret_cast<P*>(base + off); }
  static int delta_channels(const RfMixedLayer& l) { return 2 * l.kv_heads * l.dim + l.heads * l.vdim; }
  static int moe_ld(const RfMixedLayer& l) { return std::max(l.bank_inter, l.shared_inter); }
  int32_t* status() const { return base ? at<int32_t>(off_status) : nullptr; }

  void plan() {
    auto al = [](uint64_t v) { return (v + 1023) & ~uint64_t(1023); };
    const uint64_t T = (uint64_t)cfg.max_tokens, H = (uint64_t)cfg.hidden, e = esz();
    uint64_t wide = 8, mix = 8, lat = 0, rank = 0, kvw = 0, past = 0, heads = 0;
    uint64_t vfirst = 0, qout = 0, inner = 0, bc = 0, picks = 0, experts = 0, hg = 0;
    rows_ws_bytes = 0; moe_tiles = 0;
    for (const RfMixedLayer& l : layers) {
      wide = std::max<uint64_t>(wide, std::max(l.in_dim, l.inter));
      mix = std::max<uint64_t>(mix, (uint64_t)l.out_dim);
      if (l.mixer == RF_MIXER_ATTENTION) {
        vfirst = std::max<uint64_t>(vfirst, l.v_role != RF_VMIX_NONE ? (uint64_t)l.kv_heads * l.vdim : 0);
        if (l.conv_taps > 0) qout = std::max<uint64_t>(qout, (uint64_t)l.heads * l.dim);
        if (l.tensor_core) rows_ws_bytes = std::max<uint64_t>(rows_ws_bytes, rf_attn_decode_scratch_bound(l.heads, l.kv_heads, l.dim));
      }
      if (l.mixer == RF_MIXER_DELTA) inner = std::max<uint64_t>(inner, delta_channels(l));
      if (l.mixer == RF_MIXER_MAMBA1) {
        inner = std::max<uint64_t>(inner, l.inner);
        bc = std::max<uint64_t>(bc, l.dt_rank + 2 * l.states);
      }
      if (l.experts > 0) {
        picks = std::max<uint64_t>(picks, l.top + 1);
        experts = std::max<uint64_t>(experts, l.experts + l.identity + l.shared_gate);
        hg = std::max<uint64_t>(hg, moe_ld(l));
        moe_tiles = std::max(moe_tiles, l.experts + (int)(T * (l.top + 1) / 16) + 2);
      }
      if (l.mixer != RF_MIXER_LATENT_ATTENTION) continue;
      lat = std::max<uint64_t>(lat, (uint64_t)l.heads * (l.rank + l.rot_pad));
      rank = std::max<uint64_t>(rank, l.rank + l.rot_pad);
      if (l.q_rank > 0) qout = std::max<uint64_t>(qout, (uint64_t)l.heads * l.dim);
      heads = std::max<uint64_t>(heads, l.heads);
      if (l.expand_hd > 0) {
        kvw = std::max<uint64_t>(kvw, (uint64_t)l.heads * (l.expand_hd + l.vdim));
        past = std::max<uint64_t>(past, l.window > 0 ? l.window - 1 : cfg.max_seq_len);
      }
    }
    windows.clear();
    for (const RfMixedLayer& l : layers) {
      if (l.mixer != RF_MIXER_LATENT_ATTENTION || l.expand_hd <= 0) continue;
      bool known = false;
      for (const WindowPlan& w : windows) known |= w.window == l.window;
      if (!known) { windows.emplace_back(); windows.back().window = l.window; }
    }
    lat_rows = std::min<int>(cfg.max_tokens, std::max(cfg.max_seqs, 512));
    ctx_rows = (int)(T + past);
    uint64_t o = 0;
    for (int i = 0; i < 2; ++i) { off_x[i] = o; o += al(T * H * 4); }
    off_h = o; o += al(T * H * e);
    off_cast = o; o += al(T * H * e);
    off_wide = o; o += al(T * wide * e);
    off_mix = o; o += al(T * mix * e);
    off_y = o; o += al(T * H * e);
    off_side = o; o += al(T * (uint64_t)std::max(cfg.side_dim, 8) * e);
    off_qlat = o; o += al((uint64_t)lat_rows * lat * e);
    off_olat = o; o += al((uint64_t)lat_rows * lat * e);
    attn_ws_bytes = lat ? rf_latent_attn_scratch_bytes(lat_rows, (int)heads, (int)rank, cfg.max_seq_len) : 0;
    attn_ws_bytes = std::max(attn_ws_bytes, rows_ws_bytes);
    off_attn_ws = o; o += al(attn_ws_bytes);
    off_ctx = o; o += al(kvw ? (uint64_t)ctx_rows * rank * e : 0);
    off_kv = o; o += al((uint64_t)ctx_rows * kvw * e);
    off_kvmeta = o; o += al((uint64_t)cfg.max_seqs * (2 * windows.size() + 1) * sizeof(int32_t));
    off_vfirst = o; o += al(T * vfirst * e);
    off_q = o; o += al(T * qout * e);
    off_conv = o; o += al(T * inner * e);
    off_bc = o; o += al(T * bc * e);
    off_dt = o; o += al(fp32() ? 0 : T * inner * e);
    // counters, start | tile list | ids, weights, rank | slot_of, token_of_slot, slot_w (one column more)
    off_moe = o; o += al(picks ? (6 * T * picks + 2 * kMoeExperts + 4 + 4ull * moe_tiles) * 4 : 0);
    off_router = o; o += al(picks ? rf_moe_router_scratch_bytes(cfg.max_tokens, (int)experts) : 0);
    off_self = o; o += al(picks ? T * sizeof(float) : 0);
    off_xg = o; o += al(fp32() || !picks ? 0 : T * (picks - 1) * H * e);
    off_hg = o; o += al(T * picks * hg * e);
    off_yg = o; o += al(T * picks * H * e);
    off_head = o; o += al((uint64_t)std::max(cfg.max_seqs, 64) * H * e);
    argmax_bytes = rf_argmax_scratch_bytes(std::max(cfg.max_seqs, 64), cfg.vocab);
    off_argmax = o; o += al(argmax_bytes);
    const uint64_t bn = (uint64_t)((std::min(cfg.max_tokens, 256) + 15) / 16 * 16);
    sk_ws_bytes = fp32() ? 0 : (uint64_t)sm_count() * 2 * 2 * bn * 128 * sizeof(float);
    off_sk_ws = o; o += al(sk_ws_bytes);
    off_sk_flags = o; o += al(kSkFlags * sizeof(uint32_t));
    off_status = o; o += al(kStatusWords * sizeof(int32_t));
    total = o;
    planned = true;
  }
};

static HandleRegistry<MixedStack>& registry() {
  static HandleRegistry<MixedStack> r;
  return r;
}

// out[M, N] = act(x[M, K] . w[N, K]^T): the tcgen05 GEMMs for 16-bit stacks, the fp32 GEMM for 32-bit ones.
static RfGemm gemm_args(const MixedStack& s, const void* x, int64_t ldx, const void* w, void* out, int64_t ldo, int M, int N, int K, int act) {
  RfGemm g = {};
  g.x = x; g.ldx = ldx; g.w = w; g.ldw = K; g.out = out; g.ldo = ldo;
  g.M = M; g.N = N; g.K = K; g.dtype = s.cfg.dtype; g.act = act;
  if (s.fp32()) return g;
  g.w_packed = s.cfg.weights_packed;
  g.status = s.status();
  g.force_swap = -1;
  // large weights stream through the tcgen05 kernel; the latency-bound kernel keeps the small ones (side input, latents)
  g.streaming_only = (int64_t)N * K > (2 << 20);
  g.ws = s.at<float>(s.off_sk_ws); g.ws_bytes = s.sk_ws_bytes;
  g.sem = s.at<uint32_t>(s.off_sk_flags); g.sem_count = MixedStack::kSkFlags;
  return g;
}

static int linear(const MixedStack& s, const void* x, int64_t ldx, const void* w, void* out, int64_t ldo, int M, int N, int K,
                  int act, cudaStream_t st) {
  const RfGemm g = gemm_args(s, x, ldx, w, out, ldo, M, N, K, act);
  return s.fp32() ? rf_gemm_f32(&g, st) : rf_gemm(&g, st);
}

// Gated pair: weight rows of the gates, then of the ups; out[M, N] = act(gate, up) with the activation's constants.
static int linear_pair(const MixedStack& s, const void* x, int64_t ldx, const void* w, void* out, int64_t ldo, int M, int N, int K,
                       int act, float limit, float alpha, cudaStream_t st) {
  RfGemm g = gemm_args(s, x, ldx, w, out, ldo, M, N, K, act);
  g.dual_offset = N; g.act_limit = limit; g.act_alpha = alpha;
  return s.fp32() ? rf_gemm_f32(&g, st) : rf_gemm(&g, st);
}

// gelu(W_gate x) times this layer's slice of the tokens' side rows: in the GEMM's epilogue where it has one for that
static int side_gate(const MixedStack& s, const void* x, const RfMixedLayer& w, const int32_t* ids, int layer, void* out, int T, cudaStream_t st) {
  const RfMixedConfig& c = s.cfg;
  const int P = c.side_dim;
  RfGemm g = gemm_args(s, x, c.hidden, w.side_gate, out, P, T, P, c.hidden, kActGeluTanh);
  if (!s.fp32() && rf_gemm_takes_mul(&g)) {
    g.mul = (const uint8_t*)c.side_table + (size_t)layer * P * s.esz(); g.mul_row = ids; g.mul_ld = c.side_ld;
    return rf_gemm(&g, st);
  }
  int rc = s.fp32() ? rf_gemm_f32(&g, st) : rf_gemm(&g, st);
  if (rc) return rc;
  return rf_token_gate(out, P, c.side_table, c.side_ld, ids, layer * P, T, P, c.dtype, st);
}

// Rows and sequences from `seq0` / `row0` on: the same launch description for a part of the batch.
static RfRows sub_rows(const RfRows& r, int seq0, int num_seqs) {
  RfRows o = r;
  if (o.q_start) o.q_start += seq0;
  if (o.q_len) o.q_len += seq0;
  if (o.slot) o.slot += seq0;
  o.num_seqs = num_seqs;
  return o;
}

static int latent_attention(MixedStack& s, const RfMixedLayer& w, const RfMixedForward& f, const void* h, void* mix, cudaStream_t st) {
  const RfMixedConfig& c = s.cfg;
  const int T = f.tokens, H = c.hidden, QD = w.heads * w.dim, VD = w.heads * w.vdim, R = w.rank + w.rot_pad;
  const size_t e = s.esz();
  uint8_t* wide = s.at<uint8_t>(s.off_wide);
  int rc = linear(s, h, H, w.w_in, wide, w.in_dim, T, w.in_dim, H, kActNone, st);
  if (rc) return rc;
  RfLatentInsert ins = {};
  ins.norm_w = w.latent_norm; ins.pool = w.st.latent_pool; ins.rows = f.rows; ins.n_rows = T; ins.rank = w.rank; ins.rank_true = w.rank_true; ins.eps = c.eps;
  ins.rot = w.rot; ins.rot_pad = w.rot_pad; ins.cos = w.cos; ins.sin = w.sin;
  if (!w.shares) { ins.x = wide + (size_t)(w.q_rank > 0 ? w.q_rank : QD) * e; ins.ldx = w.in_dim; }
  uint8_t* queries = wide;
  int64_t ldq = w.in_dim;
  bool inserted = false;
  if (w.q_rank > 0) {
    ins.q = wide; ins.ldq = w.in_dim; ins.q_norm = w.q_latent_norm; ins.q_rank = w.q_rank; ins.q_rank_true = w.q_rank_true;
    rc = rf_latent_insert(&ins, c.dtype, st);
    if (rc) return rc;
    inserted = true;
    queries = s.at<uint8_t>(s.off_q);
    ldq = QD;
    rc = linear(s, wide, w.in_dim, w.w_uq, queries, QD, T, QD, w.q_rank, kActNone, st);
    if (rc) return rc;
  }
  RfHeadRotate turn = {};               // the rotated part of the queries; rows are filled in below
  turn.ldx = ldq; turn.xs = w.dim; turn.cos = w.cos; turn.sin = w.sin; turn.heads = w.heads; turn.dims = w.rot;
  // ---- decode rows and short portions (and everything without an expanded form): in the latent space
  const bool expand = w.expand_hd > 0 && f.short_seqs < f.rows.num_seqs;
  const int lat_total = expand ? f.short_rows : T;
  if (lat_total == 0 && !inserted) {
    rc = rf_latent_insert(&ins, c.dtype, st);
    if (rc) return rc;
  }
  for (int r0 = 0; r0 < lat_total; r0 += s.lat_rows) {
    const int n = std::min(s.lat_rows, lat_total - r0);
    RfHeadLinear q = {};
    q.x = queries + (size_t)r0 * ldq * e; q.ldx = ldq; q.xs = w.dim;
    q.y = s.at(s.off_qlat); q.ldy = (int64_t)w.heads * R; q.ys = R;
    q.w = w.w_absorb; q.rows = n; q.heads = w.heads; q.n = w.rank; q.k = w.plain; q.dtype = c.dtype;
    turn.x = (const uint8_t*)q.x + (size_t)w.plain * e; turn.y = (uint8_t*)q.y + (size_t)w.rank * e; turn.ldy = q.ldy; turn.ys = R;
    turn.pos = f.rows.pos + r0; turn.rows = n; turn.dims_pad = w.rot_pad;
    rc = rf_latent_absorb(&q, r0 == 0 && !inserted ? &ins : nullptr, w.rot > 0 ? &turn : nullptr, st);      // every row is cached before the first attends
    if (rc) return rc;
    RfLatentAttn a = {};
    a.q = s.at(s.off_qlat); a.o = s.at(s.off_olat); a.pool = w.st.latent_pool;
    a.rows = f.rows; a.rows.pos += r0;
    if (a.rows.seq_of_row) a.rows.seq_of_row += r0;
    else if (a.rows.slot) a.rows.slot += r0;
    else RF_REQUIRE(r0 == 0, "mixed stack: %d decode rows need slots", lat_total);
    a.n_rows = n; a.heads = w.heads; a.rank = R; a.vrank = w.rank; a.window = w.window; a.scale = w.scale; a.dtype = c.dtype;
    a.max_kv = w.window > 0 ? std::min(w.window, f.max_kv) : f.max_kv;
    a.ws = s.at<float>(s.off_attn_ws); a.ws_bytes = s.attn_ws_bytes;
    rc = rf_latent_attn(&a, st);
    if (rc) return rc;
    RfHeadLinear v = {};
    v.x = s.at(s.off_olat); v.ldx = (int64_t)w.heads * w.rank; v.xs = w.rank;
    v.y = (uint8_t*)mix + (size_t)r0 * VD * e; v.ldy = VD; v.ys = w.vdim;
    v.w = w.w_unabsorb; v.rows = n; v.heads = w.heads; v.n = w.vdim; v.k = w.rank; v.dtype = c.dtype;
    rc = rf_head_linear(&v, st);
    if (rc) return rc;
  }
  if (!expand) return RF_OK;
  if (w.rot > 0) {                      // their queries turn in place
    turn.x = queries + ((size_t)lat_total * ldq + w.plain) * e; turn.y = (void*)turn.x; turn.ldy = ldq; turn.ys = w.dim;
    turn.pos = f.rows.pos + lat_total; turn.rows = T - lat_total; turn.dims_pad = (w.rot + 7) / 8 * 8;
    rc = rf_head_rotate(&turn, c.dtype, st);
    if (rc) return rc;
  }
  // ---- prefill-sized portions: keys and values of the visible rows, group by group so that the buffers stay bounded
  const WindowPlan* plan = nullptr;
  for (const WindowPlan& p : s.windows)
    if (p.window == w.window) plan = &p;
  RF_REQUIRE(plan != nullptr, "mixed stack: no plan for window %d", w.window);
  for (const PortionGroup& grp : plan->groups) {
    const RfRows g = sub_rows(f.rows, f.short_seqs + grp.seq0, grp.seqs);
    const int32_t* kv_start = plan->kv_start + grp.seq0;
    const int32_t* kv_len = plan->kv_len + grp.seq0;
    void* ctx = s.at(s.off_ctx);
    uint8_t* kv = s.at<uint8_t>(s.off_kv);
    const int KD = w.heads * w.expand_hd, KV = KD + VD;
    rc = rf_latent_gather(w.st.latent_pool, ctx, &g, kv_start, kv_len, R, grp.max_len, c.dtype, st);
    if (rc) return rc;
    rc = linear(s, ctx, R, w.w_expand, kv, KV, grp.total, KV, R, kActNone, st);
    if (rc) return rc;
    RfAttn a = {};
    a.q = queries; a.ldq = ldq; a.out = mix; a.ldo = VD; a.q_rows_total = T;     // q_start holds rows of the whole batch
    a.k = kv; a.v = kv + (size_t)KD * e; a.ldk = KV; a.ldv = KV; a.kv_rows_total = grp.total;
    a.num_seqs = grp.seqs; a.Hq = w.heads; a.Hkv = w.heads; a.hd = w.expand_hd; a.vd = w.vdim;
    a.q_start = g.q_start; a.q_len = g.q_len; a.kv_start = kv_start; a.kv_len = kv_len;
    a.max_q_len = grp.max_q; a.max_kv_len = grp.max_len; a.causal = 1; a.window = w.window > 0 ? w.window : 0;
    a.scale = w.scale; a.status = s.status(); a.dtype = c.dtype;
    rc = rf_attn_prefill(&a, st);
    if (rc) return rc;
  }
  return RF_OK;
}

// Group the prefill-sized sequences of this forward per window and upload their key ranges.
static int plan_windows(MixedStack& s, const RfMixedForward& f, cudaStream_t st) {
  const int n = f.rows.num_seqs - f.short_seqs;
  if (n <= 0) return RF_OK;
  int32_t* dev = s.at<int32_t>(s.off_kvmeta);
  std::vector<int32_t> host((s.windows.size() * 2 + 1) * n);
  s.full_len = dev + s.windows.size() * 2 * n;
  s.max_full = s.max_long_q = 0;
  for (int j = 0; j < n; ++j) {
    const int q = f.h_q_len[f.short_seqs + j], len = f.h_pos0[f.short_seqs + j] + q;
    host[s.windows.size() * 2 * n + j] = len;
    s.max_full = std::max(s.max_full, len);
    s.max_long_q = std::max(s.max_long_q, q);
  }
  for (size_t i = 0; i < s.windows.size(); ++i) {
    WindowPlan& p = s.windows[i];
    int32_t* start = host.data() + i * 2 * n;
    int32_t* len = start + n;
    p.kv_start = dev + i * 2 * n; p.kv_len = p.kv_start + n;
    p.groups.clear();
    for (int j = 0; j < n; ++j) {
      const int q = f.h_q_len[f.short_seqs + j], pos0 = f.h_pos0[f.short_seqs + j];
      len[j] = (p.window > 0 ? std::min(pos0, p.window - 1) : pos0) + q;
      RF_REQUIRE(q > 0 && len[j] <= s.ctx_rows, "mixed stack: %d visible rows exceed the plan (%d)", len[j], s.ctx_rows);
      if (p.groups.empty() || p.groups.back().total + len[j] > s.ctx_rows) p.groups.push_back(PortionGroup{j, 0, 0, 0, 0});
      PortionGroup& g = p.groups.back();
      start[j] = g.total;
      ++g.seqs;
      g.total += len[j];
      g.max_len = std::max(g.max_len, (int)len[j]);
      g.max_q = std::max(g.max_q, q);
    }
  }
  RF_CUDA_CHECK(cudaMemcpyAsync(dev, host.data(), host.size() * sizeof(int32_t), cudaMemcpyHostToDevice, st));
  return RF_OK;
}

static int hgrn2(MixedStack& s, const RfMixedLayer& w, const RfMixedForward& f, const void* h, void* mix, cudaStream_t st) {
  const RfMixedConfig& c = s.cfg;
  const int T = f.tokens, H = c.hidden;
  void* wide = s.at(s.off_wide);
  int rc = linear(s, h, H, w.w_in, wide, w.in_dim, T, w.in_dim, H, kActNone, st);
  if (rc) return rc;
  RfHgrn2 a = {};
  a.x = wide; a.ldx = w.in_dim; a.f_off = w.heads * w.dim; a.v_off = 2 * w.heads * w.dim;
  a.f_bias = w.f_bias; a.lower = w.lower; a.norm_w = w.head_norm;
  a.state = w.st.rec_state; a.out = mix; a.ldo = (int64_t)w.heads * w.vdim;
  a.heads = w.heads; a.dim = w.dim; a.vdim = w.vdim; a.vdim_true = w.vdim_true; a.eps = c.eps; a.dtype = c.dtype;
  a.status = s.status();
  const bool chunked = rf_hgrn2_chunked_supported(w.dim, w.vdim, c.dtype) != 0;
  const int n_rec = chunked ? f.short_seqs : f.rows.num_seqs;
  if (n_rec > 0) {
    a.rows = sub_rows(f.rows, 0, n_rec);
    rc = rf_hgrn2_recurrent(&a, st);
    if (rc) return rc;
  }
  if (n_rec < f.rows.num_seqs) {
    a.rows = sub_rows(f.rows, n_rec, f.rows.num_seqs - n_rec);
    rc = rf_hgrn2_chunked(&a, st);
  }
  return rc;
}

static int longest_portion(const RfMixedForward& f) {
  int n = 1;
  for (int i = 0; !f.decode && i < f.rows.num_seqs; ++i) n = std::max(n, (int)f.h_q_len[i]);
  return n;
}

static int grouped_attention(MixedStack& s, const RfMixedLayer& w, const RfMixedForward& f, const void* h, void* mix, cudaStream_t st) {
  const RfMixedConfig& c = s.cfg;
  const int T = f.tokens, H = c.hidden, hd = w.dim, QD = w.heads * hd, KD = w.kv_heads * hd;
  const size_t e = s.esz();
  uint8_t* wide = s.at<uint8_t>(s.off_wide);
  int rc = linear(s, h, H, w.w_in, wide, w.in_dim, T, w.in_dim, H, kActNone, st);
  if (rc) return rc;
  RfQkvInsert q = {};
  q.qkv = wide; q.ld = w.in_dim; q.k_off = QD; q.v_off = QD + KD;
  q.q_norm = w.q_norm; q.k_norm = w.k_norm; q.cos = w.cos; q.sin = w.sin;
  q.v_first = s.at(s.off_vfirst); q.k_pool = w.st.k_pool; q.v_pool = w.st.v_pool; q.rows = f.rows;
  q.n_rows = T; q.heads = w.heads; q.kv_heads = w.kv_heads; q.hd = hd; q.dim = w.dim_true; q.vdim = w.vdim_true;
  q.rot_dims = w.rot_dims; q.v_role = w.v_role; q.v_lambda = w.v_lambda; q.eps = c.eps; q.dtype = c.dtype; q.norm_all = w.norm_all;
  q.growth = w.growth; q.growth_every = w.growth_every;
  uint8_t* queries = wide;
  int64_t ldq = w.in_dim;
  if (w.conv_taps > 0) {
    queries = s.at<uint8_t>(s.off_q);
    ldq = QD;
    q.conv_w = w.conv_w; q.conv_state = w.st.conv_state; q.q_out = queries; q.taps = w.conv_taps; q.max_q_len = longest_portion(f);
  }
  rc = rf_qkv_insert(&q, st);
  if (rc) return rc;
  RfAttn a = {};
  a.q = queries; a.ldq = ldq; a.out = mix; a.ldo = QD; a.q_rows_total = T;
  a.k_pool = w.st.k_pool; a.v_pool = w.st.v_pool; a.pool_pages = w.st.pool_pages;
  a.page_table = f.rows.page_table; a.pt_stride = f.rows.pt_stride;
  a.Hq = w.heads; a.Hkv = w.kv_heads; a.hd = hd; a.scale = w.scale; a.chunk = w.chunk; a.sink = w.sink;
  a.window = w.window; a.keep_first = w.keep_first; a.slopes = w.slopes; a.rates = w.rates;
  if (w.gated) { a.gate = wide + (size_t)(QD + 2 * KD) * e; a.ld_gate = w.in_dim; a.gate_by_head = w.gate_by_head; }
  a.status = s.status(); a.dtype = c.dtype;
  // ---- decoded rows and short portions, by row (without a tensor-core form: every row)
  const int by_row = w.tensor_core ? f.short_rows : T;
  for (int r0 = 0; r0 < by_row; r0 += 32768) {
    RfAttn b = a;
    b.num_seqs = std::min(32768, by_row - r0);
    b.q = queries + (size_t)r0 * ldq * e; b.out = (uint8_t*)mix + (size_t)r0 * QD * e;
    if (a.gate) b.gate = (const uint8_t*)a.gate + (size_t)r0 * w.in_dim * e;
    b.pos = f.rows.pos + r0; b.seq_of_row = f.rows.seq_of_row ? f.rows.seq_of_row + r0 : nullptr;
    b.slot = f.rows.slot ? f.rows.slot + (b.seq_of_row ? 0 : r0) : nullptr;
    RF_REQUIRE(r0 == 0 || b.slot, "mixed stack: %d decode rows need slots", by_row);
    b.max_kv_len = f.max_kv; b.ws = s.at<float>(s.off_attn_ws); b.ws_bytes = s.attn_ws_bytes;
    rc = w.tensor_core ? rf_attn_decode(&b, st) : rf_attn_rows(&b, st);
    if (rc) return rc;
  }
  const int n_long = f.rows.num_seqs - f.short_seqs;
  if (!w.tensor_core || n_long <= 0) return RF_OK;
  const RfRows g = sub_rows(f.rows, f.short_seqs, n_long);
  a.num_seqs = n_long; a.q_start = g.q_start; a.q_len = g.q_len; a.slot = g.slot; a.kv_len = s.full_len;
  a.max_q_len = s.max_long_q; a.max_kv_len = s.max_full; a.causal = 1;
  return rf_attn_prefill(&a, st);
}

static int mamba1(MixedStack& s, const RfMixedLayer& w, const RfMixedForward& f, const void* h, void* mix, cudaStream_t st) {
  const RfMixedConfig& c = s.cfg;
  const int T = f.tokens, H = c.hidden, BC = w.dt_rank + 2 * w.states;
  const size_t e = s.esz();
  uint8_t* wide = s.at<uint8_t>(s.off_wide);
  void* conv = s.at(s.off_conv);
  uint8_t* bc = s.at<uint8_t>(s.off_bc);
  uint8_t* dt = s.at<uint8_t>(s.off_dt);
  int rc = linear(s, h, H, w.w_in, wide, w.in_dim, T, w.in_dim, H, kActNone, st);
  if (rc) return rc;
  RfConvSilu cv = {};
  cv.x = wide; cv.ldx = w.in_dim; cv.y = conv; cv.ldy = w.inner; cv.w = w.conv_w; cv.bias = w.conv_b; cv.state = w.st.conv_state;
  cv.rows = f.rows; cv.channels = w.inner; cv.taps = w.taps; cv.dtype = c.dtype; cv.max_q_len = longest_portion(f);
  rc = rf_conv_silu(&cv, st);
  if (rc) return rc;
  rc = linear(s, conv, w.inner, w.w_x, bc, BC, T, BC, w.inner, kActNone, st);
  if (rc) return rc;
  RfMamba1 a = {};
  a.x = conv; a.ldx = w.inner; a.z = wide + (size_t)w.inner * e; a.ldz = w.in_dim; a.bc = bc; a.ld_bc = BC;
  a.dt = dt; a.ld_dt = w.inner; a.w_dt = w.w_dt_rows; a.dt_bias = w.dt_bias; a.a2 = w.a2; a.d = w.d_skip;
  a.state = w.st.rec_state; a.out = mix; a.ldo = w.inner;
  a.inner = w.inner; a.states = w.states; a.rank = w.dt_rank; a.dtype = c.dtype;
  const int n_rec = s.fp32() ? f.rows.num_seqs : f.short_seqs;
  if (n_rec > 0) {
    a.rows = sub_rows(f.rows, 0, n_rec);
    rc = rf_mamba1_recurrent(&a, st);
    if (rc) return rc;
  }
  if (n_rec < f.rows.num_seqs) {
    const int r0 = f.short_rows;
    rc = linear(s, bc + (size_t)r0 * BC * e, BC, w.w_dt, dt + (size_t)r0 * w.inner * e, w.inner, T - r0, w.inner, w.dt_rank, kActNone, st);
    if (rc) return rc;
    a.rows = sub_rows(f.rows, n_rec, f.rows.num_seqs - n_rec);
    rc = rf_mamba1_scan(&a, st);
  }
  return rc;
}

static int delta(MixedStack& s, const RfMixedLayer& w, const RfMixedForward& f, const void* h, void* mix, cudaStream_t st) {
  const RfMixedConfig& c = s.cfg;
  const int T = f.tokens, H = c.hidden, CH = MixedStack::delta_channels(w), VD = w.heads * w.vdim;
  const size_t e = s.esz();
  uint8_t* wide = s.at<uint8_t>(s.off_wide);
  int rc = linear(s, h, H, w.w_in, wide, w.in_dim, T, w.in_dim, H, kActNone, st);
  if (rc) return rc;
  RfDelta a = {};
  a.x = wide; a.ldx = w.in_dim; a.gate = wide + (size_t)CH * e; a.ldg = w.in_dim;
  a.b = wide + (size_t)(CH + VD) * e; a.a = wide + (size_t)(CH + VD + (w.heads + 7) / 8 * 8) * e; a.ld_ba = w.in_dim;
  a.rate = w.rate; a.dt_bias = w.dt_bias; a.norm_w = w.head_norm; a.state = w.st.rec_state; a.out = mix; a.ldo = VD; a.rows = f.rows;
  a.heads = w.heads; a.kv_heads = w.kv_heads; a.dim = w.dim; a.dim_true = w.dim_true; a.vdim = w.vdim; a.vdim_true = w.vdim_true; a.eps = c.eps; a.dtype = c.dtype;
  if (f.decode) {
    a.conv_w = w.conv_w; a.conv_state = w.st.conv_state; a.taps = w.taps;
    return rf_delta_recurrent(&a, st);
  }
  RfConvSilu cv = {};
  cv.x = wide; cv.ldx = w.in_dim; cv.y = s.at(s.off_conv); cv.ldy = CH; cv.w = w.conv_w; cv.state = w.st.conv_state; cv.rows = f.rows;
  cv.channels = CH; cv.taps = w.taps; cv.dtype = c.dtype; cv.max_q_len = longest_portion(f); cv.ring = 1;
  rc = rf_conv_silu(&cv, st);
  if (rc) return rc;
  a.x = cv.y; a.ldx = CH;
  const int n_rec = rf_delta_chunked_supported(w.dim, w.vdim, c.dtype) ? f.short_seqs : f.rows.num_seqs;
  if (n_rec > 0) {
    a.rows = sub_rows(f.rows, 0, n_rec);
    rc = rf_delta_recurrent(&a, st);
    if (rc) return rc;
  }
  if (n_rec < f.rows.num_seqs) {
    a.rows = sub_rows(f.rows, n_rec, f.rows.num_seqs - n_rec);
    rc = rf_delta_chunked(&a, f.short_rows, T - f.short_rows, st);
  }
  return rc;
}

// The experts' results stay where they are, one row per pick; the next stream step adds them up (see RfStreamNorm.y_slots).
static int experts(MixedStack& s, const RfMixedLayer& w, const RfMixedForward& f, const void* h, MixedStack::Pending* out, cudaStream_t st) {
  const RfMixedConfig& c = s.cfg;
  const int T = f.tokens, H = c.hidden, E = w.experts, k = w.top, pairs = T * k, has_shared = w.shared_inter > 0, cols = k + has_shared;
  const size_t e = s.esz();
  const int ldh = MixedStack::moe_ld(w), bank_rt = ceil_div(w.bank_inter, 128), kbH = ceil_div(H, 64);
  int32_t* m = s.at<int32_t>(s.off_moe);
  RfMoeRouter r = {};
  r.logits = s.at<float>(s.off_router);
  r.x = h; r.ldx = H; r.w = w.router; r.correction = w.correction; r.identity = w.identity; r.self_w = s.at<float>(s.off_self);
  r.counters = m; m += MixedStack::kMoeExperts;      // the same place whatever a layer's expert count: they are zero between launches
  r.start = m; m += MixedStack::kMoeExperts;
  r.tiles = m; m += 4 + 4 * s.moe_tiles;
  r.ids = m; m += pairs;
  r.weights = (float*)m; m += pairs;
  r.rank = m; m += pairs;
  r.slot_of = m; m += T * cols;
  r.token_of_slot = m; m += T * cols;
  r.slot_w = (float*)m;
  r.rows = T; r.experts = E + w.identity; r.width = H; r.k = k; r.groups = w.groups; r.keep = w.keep; r.score_fn = w.score_fn;
  r.norm_topk = w.norm_topk; r.scale = w.route_scale; r.slot_ld = cols; r.has_shared = has_shared; r.dtype = c.dtype;
  r.shared_gate = w.shared_gate;
  const int act = w.act == RF_MIXED_ACT_CLIPPED_GLU ? kActClippedGlu : w.act == RF_MIXED_ACT_GELU ? kActGeluErf : kActSiluMul;
  const int dual = act_is_dual(act);
  uint8_t* hg = s.at<uint8_t>(s.off_hg);
  uint8_t* yg = s.at<uint8_t>(s.off_yg);
  out->y = yg; out->slots = r.slot_of; out->picks = cols;
  if (w.identity > 0) { out->self = h; out->self_w = r.self_w; }
  if (s.fp32() || T <= MixedStack::kMoeSmallRows) {
    r.tile_rows = s.fp32() ? 64 : (pairs <= 16 * E ? 16 : 32);
    r.shared_tiles = has_shared; r.scatter = 1;
    int rc = rf_moe_router(&r, st);
    if (rc) return rc;
    RfMoeExperts x = {};
    x.tiles = r.tiles; x.experts = E; x.tile_rows = r.tile_rows; x.dtype = c.dtype;
    x.max_tiles = std::min(E, pairs) + pairs / r.tile_rows + (has_shared ? ceil_div(T, r.tile_rows) : 0);
    x.x = h; x.ldx = H; x.token_of_slot = r.token_of_slot; x.w = w.w_up; x.w_shared = w.shared_up; x.out = hg; x.ldo = ldh;
    x.n = w.inter; x.k = H; x.dual = dual; x.act = act; x.act_limit = w.act_limit; x.act_alpha = w.act_alpha; x.shared_limit = w.shared_limit;
    x.bank_section_row_tiles = E * bank_rt; x.bank_kb_total = kbH; x.rt_per_expert = bank_rt;
    if (has_shared) { x.shared_n = w.shared_inter; x.shared_k = H; x.shared_section_row_tiles = ceil_div(w.shared_inter, 128); x.shared_kb_total = kbH; }
    rc = rf_moe_experts(&x, st);
    if (rc) return rc;
    x.x = hg; x.ldx = ldh; x.token_of_slot = nullptr; x.slot_w = r.slot_w; x.w = w.w_down; x.w_shared = w.shared_down; x.out = yg; x.ldo = H;
    x.n = H; x.k = w.inter; x.dual = 0; x.act = kActNone;
    x.bank_section_row_tiles = 0; x.bank_kb_total = E * w.bank_inter / 64; x.rt_per_expert = 0; x.kb_per_expert = w.bank_inter / 64;
    if (has_shared) { x.shared_n = H; x.shared_k = w.shared_inter; x.shared_section_row_tiles = 0; x.shared_kb_total = ceil_div(w.shared_inter, 64); }
    return rf_moe_experts(&x, st);
  }
  r.tile_rows = 128;
  int rc = rf_moe_router(&r, st);
  if (rc) return rc;
  void* xg = s.at(s.off_xg);
  rc = rf_moe_gather(&r, xg, H, st);
  if (rc) return rc;
  RfMoeGroupedGemm g = {};
  g.x = xg; g.ldx = H; g.w = w.w_up; g.out = hg; g.ldo = ldh; g.tiles = r.tiles + 3; g.max_rows = pairs; g.N = w.bank_inter; g.K = H;
  g.dual = dual; g.act = act; g.act_limit = w.act_limit; g.act_alpha = w.act_alpha; g.bank_section_row_tiles = E * bank_rt; g.bank_kb_total = kbH; g.rt_per_expert = bank_rt;
  g.dtype = c.dtype; g.status = s.status();
  rc = rf_moe_grouped_gemm(&g, st);
  if (rc) return rc;
  g.x = hg; g.ldx = ldh; g.w = w.w_down; g.out = yg; g.ldo = H; g.row_scale = r.slot_w; g.N = H; g.K = w.bank_inter; g.dual = 0;
  g.act = kActNone; g.bank_section_row_tiles = 0; g.bank_kb_total = E * w.bank_inter / 64; g.rt_per_expert = 0; g.kb_per_expert = w.bank_inter / 64;
  rc = rf_moe_grouped_gemm(&g, st);
  if (rc || !has_shared) return rc;
  uint8_t* hs = hg + (size_t)pairs * ldh * e;
  rc = linear_pair(s, h, H, w.shared_up, hs, ldh, T, w.shared_inter, H, act, w.shared_limit, w.act_alpha, st);
  if (rc) return rc;
  RfGemm d = gemm_args(s, hs, ldh, w.shared_down, yg + (size_t)pairs * H * e, H, T, H, w.shared_inter, kActNone);
  if (w.shared_gate) d.row_scale = r.slot_w + pairs;
  return rf_gemm(&d, st);
}

static int forward(MixedStack& s, const RfMixedForward& f, cudaStream_t st) {
  const RfMixedConfig& c = s.cfg;
  RF_REQUIRE(s.base != nullptr, "mixed stack: arena is not bound");
  RF_REQUIRE(f.ids && f.rows.pos && f.rows.page_table, "mixed stack: ids, positions and page table are required");
  RF_REQUIRE(f.tokens >= 0 && f.tokens <= c.max_tokens, "mixed stack: %d tokens (max %d)", f.tokens, c.max_tokens);
  RF_REQUIRE(f.rows.num_seqs > 0 && f.rows.num_seqs <= c.max_seqs, "mixed stack: %d sequences (max %d)", f.rows.num_seqs, c.max_seqs);
  if (f.decode) RF_REQUIRE(f.tokens == f.rows.num_seqs && f.short_seqs == f.tokens, "mixed stack: a decode step has one row per sequence");
  else RF_REQUIRE(f.rows.seq_of_row && f.rows.q_start && f.rows.q_len, "mixed stack: portions need seq_of_row, q_start and q_len");
  if (!f.decode) RF_REQUIRE(f.h_q_len && f.h_pos0, "mixed stack: portions need the host arrays");
  if (f.tokens == 0) return RF_OK;
  int rc = plan_windows(s, f, st);
  if (rc) return rc;
  const int T = f.tokens, H = c.hidden;
  void* h = s.at(s.off_h);
  void* cast = s.at(s.off_cast);
  void* mix = s.at(s.off_mix);
  void* y = s.at(s.off_y);
  void* side = s.at(s.off_side);
  int cur = -1;                       // stream buffer in use; -1: still the embedding
  MixedStack::Pending pend;           // sublayer output that the next stream_norm adds
  // stream step: adds the pending output, optionally writes the 16-bit copy and / or the normalised rows
  auto step = [&](const float* norm_w, const float* shift, float* shift_state, bool want_cast, const float* conv_w = nullptr, void* conv_state = nullptr) -> int {
    RfStreamNorm a = {};
    a.x = cur < 0 ? nullptr : s.at<float>(s.off_x[cur]);
    a.table = c.embed; a.ids = f.ids; a.embed_scale = c.embed_scale; a.y_mult = c.residual_mult;
    if (cur < 0 && c.pair_table) {
      a.table2 = c.pair_table; a.last_token = s.layers[0].st.last_token; a.buckets = c.pair_buckets;
      a.mul_prev = c.pair_mul_prev; a.mul_cur = c.pair_mul_cur;
    }
    a.y = pend.y; a.y_norm_w = pend.norm; a.y_slots = pend.slots; a.y_picks = pend.picks; a.y_self = pend.self; a.y_self_w = pend.self_w;
    const int nxt = cur < 0 ? 0 : cur ^ 1;
    a.x_out = s.at<float>(s.off_x[nxt]);
    a.x_cast = want_cast ? cast : nullptr;
    a.norm_w = norm_w; a.out = norm_w ? h : nullptr; a.shift = shift; a.shift_state = shift_state;
    a.rows = f.rows; a.n_rows = T; a.H = H; a.dim = c.hidden_true; a.eps = c.eps; a.dtype = c.dtype;
    cur = nxt;
    pend = {};
    if (!conv_w) return rf_stream_norm(&a, st);
    if (f.decode && !s.fp32() && H <= 8192) {
      a.conv_w = conv_w; a.conv_state = conv_state; a.conv_taps = c.input_taps;
      return rf_stream_norm(&a, st);
    }
    a.out = cast;                       // portions: the rows are written, then convolved
    int rc = rf_stream_norm(&a, st);
    if (rc) return rc;
    RfConvSilu cv = {};
    cv.x = cast; cv.ldx = H; cv.y = h; cv.ldy = H; cv.w = conv_w; cv.state = conv_state; cv.rows = f.rows;
    cv.channels = H; cv.taps = c.input_taps; cv.dtype = c.dtype; cv.max_q_len = longest_portion(f); cv.add = 1;
    return rf_conv_silu(&cv, st);
  };
  for (int l = 0; l < c.layers; ++l) {
    const RfMixedLayer& w = s.layers[l];
    rc = c.norm_after ? step(nullptr, nullptr, nullptr, true) : step(w.norm1, w.shift, w.st.shift_state, false, w.input_conv[0], w.st.input_state[0]);
    if (rc) return rc;
    const void* in = c.norm_after ? cast : h;
    switch (w.mixer) {
      case RF_MIXER_LATENT_ATTENTION: rc = latent_attention(s, w, f, in, mix, st); break;
      case RF_MIXER_HGRN2: rc = hgrn2(s, w, f, in, mix, st); break;
      case RF_MIXER_DELTA: rc = delta(s, w, f, in, mix, st); break;
      case RF_MIXER_ATTENTION: rc = grouped_attention(s, w, f, in, mix, st); break;
      default: rc = mamba1(s, w, f, in, mix, st);
    }
    if (rc) return rc;
    rc = linear(s, mix, w.out_dim, w.w_o, y, H, T, H, w.out_dim, kActNone, st);
    if (rc) return rc;
    pend.y = y; pend.norm = c.norm_after ? w.norm1 : w.norm1b;
    if (w.inter > 0) {
      rc = c.norm_after ? step(nullptr, nullptr, nullptr, true) : step(w.norm2, nullptr, nullptr, false, w.input_conv[1], w.st.input_state[1]);
      if (rc) return rc;
      if (w.experts > 0) {
        rc = experts(s, w, f, in, &pend, st);
      } else {
        void* wide = s.at(s.off_wide);
        rc = w.act != RF_MIXED_ACT_RELU2
                 ? linear_pair(s, in, H, w.w_up, wide, w.inter, T, w.inter, H, w.act == RF_MIXED_ACT_SWIGLU ? kActSiluMul : kActClippedGlu, w.act_limit, w.act_alpha, st)
                 : linear(s, in, H, w.w_up, wide, w.inter, T, w.inter, H, kActRelu2, st);
        if (rc) return rc;
        rc = linear(s, wide, w.inter, w.w_down, y, H, T, H, w.inter, kActNone, st);
        pend.y = y;
      }
      if (rc) return rc;
      pend.norm = c.norm_after ? w.norm2 : w.norm2b;
    }
    if (c.side_dim > 0) {
      rc = step(nullptr, nullptr, nullptr, true);
      if (rc) return rc;
      const int P = c.side_dim;
      rc = side_gate(s, cast, w, f.ids, l, side, T, st);
      if (rc) return rc;
      rc = linear(s, side, P, w.side_proj, y, H, T, H, P, kActNone, st);
      if (rc) return rc;
      pend.y = y; pend.norm = w.side_norm;
    }
    if (f.taps) {
      RfStreamNorm a = {};
      a.x = s.at<float>(s.off_x[cur]); a.y_mult = c.residual_mult; a.y = pend.y; a.y_norm_w = pend.norm; a.y_slots = pend.slots; a.y_picks = pend.picks;
      a.y_self = pend.self; a.y_self_w = pend.self_w;
      a.x_out = f.taps + (size_t)l * T * H;
      a.rows = f.rows; a.n_rows = T; a.H = H; a.dim = c.hidden_true; a.eps = c.eps; a.dtype = c.dtype;
      rc = rf_stream_norm(&a, st);
      if (rc) return rc;
    }
  }
  s.cur = cur;
  s.tail = pend;
  return RF_OK;
}

}  // namespace rf

using namespace rf;

#define RF_GET_MIXED(h)                                                                    \
  std::shared_ptr<MixedStack> sp = registry().get(h);                                      \
  if (!sp) return fail(RF_ERR_BAD_ARG, "unknown mixed-stack handle %lld", (long long)(h)); \
  MixedStack& s = *sp;

extern "C" int64_t rf_mixed_create(const RfMixedConfig* c) {
  if (!c || c->layers <= 0 || c->hidden <= 0 || c->hidden % 8 || c->hidden_true <= 0 || c->hidden_true > c->hidden || c->vocab <= 0 ||
      c->vocab_ld < c->vocab || c->vocab_ld % 8 || c->dtype < 0 || c->dtype > 2 || c->max_tokens <= 0 || c->max_seqs <= 0 ||
      c->max_seq_len <= 0 || c->side_dim < 0 || c->side_dim % 8 || !c->embed || !c->final_norm || !c->w_lm || c->long_min < 1 ||
      (c->dtype == kF32 && c->weights_packed) || c->logit_softcap < 0.f || c->input_taps < 0 || (c->input_taps > 0 && c->norm_after) ||
      (c->pair_table && (c->pair_buckets <= 0 || c->pair_mul_prev < 0 || c->pair_mul_cur < 0))) {
    fail(RF_ERR_BAD_ARG, "invalid mixed-stack config");
    return -1;
  }
  auto s = std::make_unique<MixedStack>();
  s->cfg = *c;
  s->layers.resize(c->layers);
  return registry().insert(std::move(s));
}

extern "C" int rf_mixed_destroy(int64_t h) {
  return registry().erase(h) ? RF_OK : fail(RF_ERR_BAD_ARG, "unknown mixed-stack handle %lld", (long long)h);
}

extern "C" int rf_mixed_set_layer(int64_t h, int32_t layer, const RfMixedLayer* w) {
  RF_GET_MIXED(h);
  RF_REQUIRE(w && layer >= 0 && layer < s.cfg.layers, "layer index %d out of range", layer);
  RF_REQUIRE(w->in_dim % 8 == 0 && w->out_dim > 0 && w->out_dim % 8 == 0 && w->inter >= 0 && w->inter % 8 == 0, "layer %d: projection and feed-forward sizes", layer);
  if (s.cfg.input_taps > 0)
    RF_REQUIRE(w->input_conv[0] && !w->shift && (w->inter == 0 || w->input_conv[1]) && (s.cfg.input_taps == 1 || (w->st.input_state[0] && w->st.input_state[1])),
               "layer %d: input convolutions", layer);
  if (w->mixer != RF_MIXER_MAMBA1) {
    RF_REQUIRE(w->heads > 0 && w->dim > 0 && w->dim % 8 == 0 && w->vdim > 0 && w->vdim % 8 == 0, "layer %d: head sizes", layer);
    RF_REQUIRE(w->out_dim == w->heads * w->vdim, "layer %d: output projection columns", layer);
  }
  RF_REQUIRE(w->norm1 && w->w_in && w->w_o && (!w->shift || w->st.shift_state), "layer %d: missing weights", layer);
  if (w->inter > 0) RF_REQUIRE(w->norm2 && w->w_up && w->w_down && (w->act == RF_MIXED_ACT_RELU2 || w->act == RF_MIXED_ACT_SWIGLU ||
                                  (w->act == RF_MIXED_ACT_CLIPPED_GLU && w->act_limit > 0.f) || (w->act == RF_MIXED_ACT_GELU && w->experts > 0 && w->shared_inter == 0)),
                                 "layer %d: feed-forward weights", layer);
  if (s.cfg.pair_table) RF_REQUIRE(w->st.last_token && !w->shift, "layer %d: token pairs need the carried tokens and no token shift", layer);
  if (w->experts > 0) {
    const int routed = w->experts + w->identity;
    RF_REQUIRE(w->inter > 0 && w->router && w->identity >= 0 && routed <= 256 && w->top > 0 && w->top <= 32 && w->groups > 0 && routed % w->groups == 0 &&
                   w->keep > 0 && w->keep <= w->groups && w->top <= routed / w->groups * w->keep,
               "layer %d: %d experts in %d groups, %d kept, %d chosen", layer, w->experts, w->groups, w->keep, w->top);
    RF_REQUIRE(w->bank_inter >= w->inter && w->bank_inter % (s.cfg.dtype == kF32 ? 8 : 128) == 0 && w->shared_inter >= 0 && w->shared_inter % 8 == 0 &&
                   (w->shared_inter == 0 || (w->shared_up && w->shared_down)) && (!w->shared_gate || w->shared_inter > 0) &&
                   (w->act != RF_MIXED_ACT_CLIPPED_GLU || w->shared_inter == 0 || w->shared_limit > 0.f), "layer %d: expert widths", layer);
    RF_REQUIRE(s.cfg.dtype == kF32 || s.cfg.weights_packed, "layer %d: experts need tile-major weights", layer);
  }
  if (w->mixer == RF_MIXER_LATENT_ATTENTION) {
    RF_REQUIRE(w->rank > 0 && w->rank % 16 == 0 && w->rank_true > 0 && (w->latent_norm || w->shares) && w->w_absorb && w->w_unabsorb && w->st.latent_pool,
               "layer %d: latent-attention weights", layer);
    RF_REQUIRE(w->q_rank % 8 == 0 && (w->q_rank == 0 || (w->w_uq && w->q_latent_norm && w->q_rank_true > 0 && w->q_rank_true <= w->q_rank)) && (!w->shares || w->q_rank > 0),
               "layer %d: query latent", layer);
    RF_REQUIRE(w->plain > 0 && w->plain % 8 == 0 && w->rot >= 0 && w->rot % 2 == 0 && w->rot_pad >= w->rot && w->rot_pad % 16 == 0 &&
                   w->plain + (w->rot + 7) / 8 * 8 <= w->dim && (w->rot == 0 || (w->cos && w->sin)), "layer %d: rotated part", layer);
    RF_REQUIRE(w->in_dim >= (w->q_rank > 0 ? w->q_rank : w->heads * w->dim) + (w->shares ? 0 : w->rank + w->rot_pad), "layer %d: input projection rows", layer);
    RF_REQUIRE(w->expand_hd == 0 || (w->w_expand && w->dim == w->expand_hd && (w->vdim == w->expand_hd || (w->expand_hd == 192 && w->vdim == 128)) && s.cfg.dtype != kF32),
               "layer %d: expanded heads", layer);
  } else if (w->mixer == RF_MIXER_ATTENTION) {
    RF_REQUIRE(w->dim == w->vdim && w->kv_heads > 0 && w->heads % w->kv_heads == 0 && w->dim_true > 0 && w->dim_true <= w->dim &&
                   w->vdim_true > 0 && w->vdim_true <= w->vdim && w->st.k_pool && w->st.v_pool && w->st.pool_pages > 0, "layer %d: attention", layer);
    RF_REQUIRE(w->in_dim >= (w->heads + 2 * w->kv_heads) * w->dim + (w->gated ? w->heads * (w->gate_by_head ? 1 : w->dim) : 0), "layer %d: input projection rows", layer);
    RF_REQUIRE(w->conv_taps >= 0 && (w->conv_taps == 0 || (w->conv_w && !w->norm_all && (w->conv_taps == 1 || w->st.conv_state))) && w->keep_first >= 0,
               "layer %d: convolution of %d taps, %d kept positions", layer, w->conv_taps, w->keep_first);
    RF_REQUIRE(!w->tensor_core || (s.cfg.dtype != kF32 && (w->dim == 64 || w->dim == 128 || w->dim == 256) && w->scale > 0.f), "layer %d: heads", layer);
    RF_REQUIRE(w->rot_dims % 2 == 0 && w->rot_dims >= 0 && w->rot_dims <= w->dim_true && (w->rot_dims == 0 || (w->cos && w->sin)), "layer %d: rotation", layer);
  } else if (w->mixer == RF_MIXER_DELTA) {
    RF_REQUIRE(w->kv_heads > 0 && w->heads % w->kv_heads == 0 && w->dim_true > 0 && w->dim_true <= w->dim && w->vdim_true > 0 && w->vdim_true <= w->vdim &&
                   w->taps > 0 && w->in_dim >= MixedStack::delta_channels(*w) + w->heads * w->vdim + 2 * ((w->heads + 7) / 8 * 8), "layer %d: delta-rule sizes", layer);
    RF_REQUIRE(w->conv_w && w->rate && w->dt_bias && w->head_norm && w->st.rec_state && w->st.conv_state, "layer %d: delta-rule weights", layer);
  } else if (w->mixer == RF_MIXER_MAMBA1) {
    RF_REQUIRE(w->inner > 0 && w->inner % 8 == 0 && w->states > 0 && w->states % 8 == 0 && w->states <= 256 && w->dt_rank > 0 && w->dt_rank % 8 == 0 &&
                   w->taps > 0 && w->in_dim == 2 * w->inner && w->out_dim == w->inner, "layer %d: scan sizes", layer);
    RF_REQUIRE(w->conv_w && w->a2 && w->d_skip && w->dt_bias && w->w_x && w->w_dt && w->w_dt_rows && w->st.rec_state && (w->taps == 1 || w->st.conv_state),
               "layer %d: scan weights", layer);
  } else {
    RF_REQUIRE(w->mixer == RF_MIXER_HGRN2 && w->f_bias && w->lower && w->head_norm && w->st.rec_state, "layer %d: HGRN2 weights", layer);
    RF_REQUIRE(w->in_dim >= w->heads * (2 * w->dim + w->vdim), "layer %d: input projection rows", layer);
  }
  if (s.cfg.side_dim > 0) RF_REQUIRE(s.cfg.side_table && w->side_gate && w->side_proj && w->side_norm, "layer %d: side-input weights", layer);
  s.layers[layer] = *w;
  s.planned = false;
  return RF_OK;
}

extern "C" int rf_mixed_set_state(int64_t h, int32_t layer, const RfMixedState* st) {
  RF_GET_MIXED(h);
  RF_REQUIRE(st && layer >= 0 && layer < s.cfg.layers, "layer index %d out of range", layer);
  s.layers[layer].st = *st;
  return RF_OK;
}

extern "C" int rf_mixed_set_rotation(int64_t h, int32_t layer, const float* cos, const float* sin) {
  RF_GET_MIXED(h);
  RF_REQUIRE(cos && sin && layer >= 0 && layer < s.cfg.layers, "rotation tables of layer %d", layer);
  s.layers[layer].cos = cos;
  s.layers[layer].sin = sin;
  return RF_OK;
}

extern "C" int rf_mixed_set_context(int64_t h, int32_t max_seq_len) {
  RF_GET_MIXED(h);
  RF_REQUIRE(max_seq_len > 0, "mixed stack: context of %d tokens", max_seq_len);
  s.cfg.max_seq_len = std::max(s.cfg.max_seq_len, max_seq_len);
  s.planned = false;
  s.base = nullptr;
  return RF_OK;
}

extern "C" uint64_t rf_mixed_arena_bytes(int64_t h) {
  std::shared_ptr<MixedStack> sp = registry().get(h);
  if (!sp) return 0;
  sp->plan();
  return sp->total;
}

extern "C" int rf_mixed_bind_arena(int64_t h, void* base, uint64_t bytes) {
  RF_GET_MIXED(h);
  RF_REQUIRE(s.planned, "mixed stack: query rf_mixed_arena_bytes after the last layer is set");
  RF_REQUIRE(base && bytes >= s.total && (reinterpret_cast<uintptr_t>(base) & 1023) == 0, "mixed stack: arena of %llu B (plan %llu B)",
             (unsigned long long)bytes, (unsigned long long)s.total);
  s.base = static_cast<uint8_t*>(base);
  return RF_OK;
}

extern "C" int32_t* rf_mixed_status_ptr(int64_t h) {
  std::shared_ptr<MixedStack> sp = registry().get(h);
  return sp ? sp->status() : nullptr;
}

extern "C" int rf_mixed_forward(int64_t h, const RfMixedForward* f, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_GET_MIXED(h);
  RF_REQUIRE(f != nullptr, "null forward args");
  return forward(s, *f, static_cast<cudaStream_t>(stream));
}

extern "C" int rf_mixed_head(int64_t h, const int32_t* row_idx, int32_t rows, int32_t* out_ids, float* out_vals, void* logits,
                             rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_GET_MIXED(h);
  const RfMixedConfig& c = s.cfg;
  RF_REQUIRE(s.base && logits, "mixed stack: logits buffer");
  RF_REQUIRE(rows > 0 && rows <= std::max(c.max_seqs, 64), "head rows %d (max %d)", rows, std::max(c.max_seqs, 64));
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  RfStreamNorm a = {};
  a.x = s.at<float>(s.off_x[s.cur]); a.row_idx = row_idx; a.y_mult = c.residual_mult;
  a.y = s.tail.y; a.y_norm_w = s.tail.norm; a.y_slots = s.tail.slots; a.y_picks = s.tail.picks; a.y_self = s.tail.self; a.y_self_w = s.tail.self_w;
  a.norm_w = c.final_norm; a.out = s.at(s.off_head);
  a.n_rows = rows; a.H = c.hidden; a.dim = c.hidden_true; a.eps = c.eps; a.dtype = c.dtype;
  int rc = rf_stream_norm(&a, st);
  if (rc) return rc;
  RfGemm g = gemm_args(s, s.at(s.off_head), c.hidden, c.w_lm, logits, c.vocab_ld, rows, c.vocab_ld, c.hidden, c.logit_softcap > 0.f ? kActSoftCap : kActNone);
  g.act_limit = c.logit_softcap;
  rc = s.fp32() ? rf_gemm_f32(&g, st) : rf_gemm(&g, st);
  if (rc) return rc;
  if (out_ids)
    rc = rf_argmax(logits, rows, c.vocab, c.vocab_ld, out_ids, out_vals, 0, s.at(s.off_argmax), s.argmax_bytes, c.dtype, st);
  return rc;
}

extern "C" void rf_mixed_struct_sizes(int32_t* out) {
  out[0] = (int32_t)sizeof(RfMixedConfig); out[1] = (int32_t)sizeof(RfMixedLayer); out[2] = (int32_t)sizeof(RfMixedForward);
  out[3] = (int32_t)sizeof(RfRows); out[4] = (int32_t)sizeof(RfStreamNorm); out[5] = (int32_t)sizeof(RfLatentAttn);
  out[6] = (int32_t)sizeof(RfHgrn2); out[7] = (int32_t)sizeof(RfHeadLinear); out[8] = (int32_t)sizeof(RfMixedState);
  out[9] = (int32_t)sizeof(RfAttn); out[10] = (int32_t)sizeof(RfQkvInsert); out[11] = (int32_t)sizeof(RfConvSilu);
  out[15] = (int32_t)sizeof(RfLatentInsert); out[16] = (int32_t)sizeof(RfHeadRotate); out[17] = (int32_t)sizeof(RfDelta);
  out[12] = (int32_t)sizeof(RfMamba1); out[13] = (int32_t)sizeof(RfMoeRouter); out[14] = (int32_t)sizeof(RfMoeExperts);
}
