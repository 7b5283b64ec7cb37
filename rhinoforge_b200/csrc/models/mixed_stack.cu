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
           off_status = 0, total = 0;
  uint64_t attn_ws_bytes = 0, argmax_bytes = 0, sk_ws_bytes = 0;
  int lat_rows = 0;       // rows one latent-space attention launch takes
  int ctx_rows = 0;       // rows of expanded keys / values one group of portions takes
  int cur = 0;            // which stream buffer holds the last forward's rows
  bool side_pending = false;
  bool planned = false;
  static constexpr int kSkFlags = 1024;

  size_t esz() const { return cfg.dtype == kF32 ? 4 : 2; }
  bool fp32() const { return cfg.dtype == kF32; }
  template <typename P = void> P* at(uint64_t off) const { return reinterpret_cast<P*>(base + off); }
  int32_t* status() const { return base ? at<int32_t>(off_status) : nullptr; }

  void plan() {
    auto al = [](uint64_t v) { return (v + 1023) & ~uint64_t(1023); };
    const uint64_t T = (uint64_t)cfg.max_tokens, H = (uint64_t)cfg.hidden, e = esz();
    uint64_t wide = 8, mix = 8, lat = 0, rank = 0, kvw = 0, past = 0, heads = 0;
    for (const RfMixedLayer& l : layers) {
      wide = std::max<uint64_t>(wide, std::max(l.in_dim, l.inter));
      mix = std::max<uint64_t>(mix, (uint64_t)l.heads * l.vdim);
      if (l.mixer != RF_MIXER_LATENT_ATTENTION) continue;
      lat = std::max<uint64_t>(lat, (uint64_t)l.heads * l.rank);
      rank = std::max<uint64_t>(rank, l.rank);
      heads = std::max<uint64_t>(heads, l.heads);
      if (l.expand_hd > 0) {
        kvw = std::max<uint64_t>(kvw, 2ull * l.heads * l.expand_hd);
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
    off_attn_ws = o; o += al(attn_ws_bytes);
    off_ctx = o; o += al(kvw ? (uint64_t)ctx_rows * rank * e : 0);
    off_kv = o; o += al((uint64_t)ctx_rows * kvw * e);
    off_kvmeta = o; o += al((uint64_t)cfg.max_seqs * 2 * windows.size() * sizeof(int32_t));
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
  const int T = f.tokens, H = c.hidden, QD = w.heads * w.dim, VD = w.heads * w.vdim;
  const size_t e = s.esz();
  uint8_t* wide = s.at<uint8_t>(s.off_wide);
  int rc = linear(s, h, H, w.w_in, wide, w.in_dim, T, w.in_dim, H, kActNone, st);
  if (rc) return rc;
  RfLatentInsert ins = {wide + (size_t)QD * e, w.in_dim, w.latent_norm, w.latent_pool, f.rows, T, w.rank, w.rank_true, c.eps};
  // ---- decode rows and short portions (and everything without an expanded form): in the latent space
  const bool expand = w.expand_hd > 0 && f.short_seqs < f.rows.num_seqs;
  const int lat_total = expand ? f.short_rows : T;
  if (lat_total == 0) {
    rc = rf_latent_insert(ins.x, ins.ldx, ins.norm_w, ins.pool, &ins.rows, T, w.rank, w.rank_true, c.eps, c.dtype, st);
    if (rc) return rc;
  }
  for (int r0 = 0; r0 < lat_total; r0 += s.lat_rows) {
    const int n = std::min(s.lat_rows, lat_total - r0);
    RfHeadLinear q = {};
    q.x = wide + (size_t)r0 * w.in_dim * e; q.ldx = w.in_dim; q.xs = w.dim;
    q.y = s.at(s.off_qlat); q.ldy = (int64_t)w.heads * w.rank; q.ys = w.rank;
    q.w = w.w_absorb; q.rows = n; q.heads = w.heads; q.n = w.rank; q.k = w.dim; q.dtype = c.dtype;
    rc = r0 == 0 ? rf_latent_absorb(&q, &ins, st) : rf_head_linear(&q, st);      // every row is cached before the first attends
    if (rc) return rc;
    RfLatentAttn a = {};
    a.q = s.at(s.off_qlat); a.o = s.at(s.off_olat); a.pool = w.latent_pool;
    a.rows = f.rows; a.rows.pos += r0;
    if (a.rows.seq_of_row) a.rows.seq_of_row += r0;
    else if (a.rows.slot) a.rows.slot += r0;
    else RF_REQUIRE(r0 == 0, "mixed stack: %d decode rows need slots", lat_total);
    a.n_rows = n; a.heads = w.heads; a.rank = w.rank; a.window = w.window; a.scale = w.scale; a.dtype = c.dtype;
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
    const int KD = w.heads * w.expand_hd, KV = 2 * KD;
    rc = rf_latent_gather(w.latent_pool, ctx, &g, kv_start, kv_len, w.rank, grp.max_len, c.dtype, st);
    if (rc) return rc;
    rc = linear(s, ctx, w.rank, w.w_expand, kv, KV, grp.total, KV, w.rank, kActNone, st);
    if (rc) return rc;
    RfAttn a = {};
    a.q = wide; a.ldq = w.in_dim; a.out = mix; a.ldo = VD; a.q_rows_total = T;     // q_start holds rows of the whole batch
    a.k = kv; a.v = kv + (size_t)KD * e; a.ldk = KV; a.ldv = KV; a.kv_rows_total = grp.total;
    a.num_seqs = grp.seqs; a.Hq = w.heads; a.Hkv = w.heads; a.hd = w.expand_hd;
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
  if (n <= 0 || s.windows.empty()) return RF_OK;
  int32_t* dev = s.at<int32_t>(s.off_kvmeta);
  std::vector<int32_t> host((size_t)s.windows.size() * 2 * n);
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
  a.state = w.rec_state; a.out = mix; a.ldo = (int64_t)w.heads * w.vdim;
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

static int forward(MixedStack& s, const RfMixedForward& f, cudaStream_t st) {
  const RfMixedConfig& c = s.cfg;
  RF_REQUIRE(s.base != nullptr, "mixed stack: arena is not bound");
  RF_REQUIRE(f.ids && f.rows.pos && f.rows.page_table, "mixed stack: ids, positions and page table are required");
  RF_REQUIRE(f.tokens >= 0 && f.tokens <= c.max_tokens, "mixed stack: %d tokens (max %d)", f.tokens, c.max_tokens);
  RF_REQUIRE(f.rows.num_seqs > 0 && f.rows.num_seqs <= c.max_seqs, "mixed stack: %d sequences (max %d)", f.rows.num_seqs, c.max_seqs);
  if (f.decode) RF_REQUIRE(f.tokens == f.rows.num_seqs && f.short_seqs == f.tokens, "mixed stack: a decode step has one row per sequence");
  else RF_REQUIRE(f.rows.seq_of_row && f.rows.q_start && f.rows.q_len, "mixed stack: portions need seq_of_row, q_start and q_len");
  if (f.short_seqs < f.rows.num_seqs) RF_REQUIRE(f.h_q_len && f.h_pos0, "mixed stack: portions need the host arrays");
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
  const void* pend = nullptr;         // sublayer output that the next stream_norm adds
  const float* pend_norm = nullptr;
  // stream step: adds the pending output, optionally writes the 16-bit copy and / or the normalised rows
  auto step = [&](const float* norm_w, const float* shift, float* shift_state, bool want_cast) -> int {
    RfStreamNorm a = {};
    a.x = cur < 0 ? nullptr : s.at<float>(s.off_x[cur]);
    a.table = c.embed; a.ids = f.ids;
    a.y = pend; a.y_norm_w = pend_norm;
    const int nxt = cur < 0 ? 0 : cur ^ 1;
    a.x_out = s.at<float>(s.off_x[nxt]);
    a.x_cast = want_cast ? cast : nullptr;
    a.norm_w = norm_w; a.out = norm_w ? h : nullptr; a.shift = shift; a.shift_state = shift_state;
    a.rows = f.rows; a.n_rows = T; a.H = H; a.dim = c.hidden_true; a.eps = c.eps; a.dtype = c.dtype;
    cur = nxt;
    pend = nullptr; pend_norm = nullptr;
    return rf_stream_norm(&a, st);
  };
  for (int l = 0; l < c.layers; ++l) {
    const RfMixedLayer& w = s.layers[l];
    rc = step(w.norm1, w.shift, w.shift_state, false);
    if (rc) return rc;
    rc = w.mixer == RF_MIXER_LATENT_ATTENTION ? latent_attention(s, w, f, h, mix, st) : hgrn2(s, w, f, h, mix, st);
    if (rc) return rc;
    const int MD = w.heads * w.vdim;
    rc = linear(s, mix, MD, w.w_o, y, H, T, H, MD, kActNone, st);
    if (rc) return rc;
    pend = y;
    if (w.inter > 0) {
      rc = step(w.norm2, nullptr, nullptr, false);
      if (rc) return rc;
      void* wide = s.at(s.off_wide);
      rc = linear(s, h, H, w.w_up, wide, w.inter, T, w.inter, H, kActRelu2, st);
      if (rc) return rc;
      rc = linear(s, wide, w.inter, w.w_down, y, H, T, H, w.inter, kActNone, st);
      if (rc) return rc;
      pend = y;
    }
    if (c.side_dim > 0) {
      rc = step(nullptr, nullptr, nullptr, true);
      if (rc) return rc;
      const int P = c.side_dim;
      rc = side_gate(s, cast, w, f.ids, l, side, T, st);
      if (rc) return rc;
      rc = linear(s, side, P, w.side_proj, y, H, T, H, P, kActNone, st);
      if (rc) return rc;
      pend = y; pend_norm = w.side_norm;
    }
    if (f.taps) {
      RfStreamNorm a = {};
      a.x = s.at<float>(s.off_x[cur]); a.y = pend; a.y_norm_w = pend_norm;
      a.x_out = f.taps + (size_t)l * T * H;
      a.rows = f.rows; a.n_rows = T; a.H = H; a.dim = c.hidden_true; a.eps = c.eps; a.dtype = c.dtype;
      rc = rf_stream_norm(&a, st);
      if (rc) return rc;
    }
  }
  s.cur = cur;
  s.side_pending = c.side_dim > 0;
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
      (c->dtype == kF32 && c->weights_packed)) {
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
  RF_REQUIRE(w->heads > 0 && w->dim > 0 && w->dim % 8 == 0 && w->vdim > 0 && w->vdim % 8 == 0 && w->in_dim % 8 == 0 &&
                 w->inter >= 0 && w->inter % 8 == 0, "layer %d: head and feed-forward sizes", layer);
  RF_REQUIRE(w->norm1 && w->w_in && w->w_o && (!w->shift || w->shift_state), "layer %d: missing weights", layer);
  if (w->inter > 0) RF_REQUIRE(w->norm2 && w->w_up && w->w_down && w->act == RF_MIXED_ACT_RELU2, "layer %d: feed-forward weights", layer);
  if (w->mixer == RF_MIXER_LATENT_ATTENTION) {
    RF_REQUIRE(w->rank > 0 && w->rank % 16 == 0 && w->rank_true > 0 && w->latent_norm && w->w_absorb && w->w_unabsorb && w->latent_pool,
               "layer %d: latent-attention weights", layer);
    RF_REQUIRE(w->in_dim >= w->heads * w->dim + w->rank, "layer %d: input projection rows", layer);
    RF_REQUIRE(w->expand_hd == 0 || (w->w_expand && w->dim == w->expand_hd && w->vdim == w->expand_hd && s.cfg.dtype != kF32),
               "layer %d: expanded heads", layer);
  } else {
    RF_REQUIRE(w->mixer == RF_MIXER_HGRN2 && w->f_bias && w->lower && w->head_norm && w->rec_state, "layer %d: HGRN2 weights", layer);
    RF_REQUIRE(w->in_dim >= w->heads * (2 * w->dim + w->vdim), "layer %d: input projection rows", layer);
  }
  if (s.cfg.side_dim > 0) RF_REQUIRE(s.cfg.side_table && w->side_gate && w->side_proj && w->side_norm, "layer %d: side-input weights", layer);
  s.layers[layer] = *w;
  s.planned = false;
  return RF_OK;
}

extern "C" int rf_mixed_set_state(int64_t h, int32_t layer, void* latent_pool, float* rec_state, float* shift_state) {
  RF_GET_MIXED(h);
  RF_REQUIRE(layer >= 0 && layer < s.cfg.layers, "layer index %d out of range", layer);
  if (latent_pool) s.layers[layer].latent_pool = latent_pool;
  if (rec_state) s.layers[layer].rec_state = rec_state;
  if (shift_state) s.layers[layer].shift_state = shift_state;
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
  a.x = s.at<float>(s.off_x[s.cur]); a.row_idx = row_idx;
  if (s.side_pending) { a.y = s.at(s.off_y); a.y_norm_w = s.layers[c.layers - 1].side_norm; }
  else a.y = s.at(s.off_y);
  a.norm_w = c.final_norm; a.out = s.at(s.off_head);
  a.n_rows = rows; a.H = c.hidden; a.dim = c.hidden_true; a.eps = c.eps; a.dtype = c.dtype;
  int rc = rf_stream_norm(&a, st);
  if (rc) return rc;
  rc = linear(s, s.at(s.off_head), c.hidden, c.w_lm, logits, c.vocab_ld, rows, c.vocab_ld, c.hidden, kActNone, st);
  if (rc) return rc;
  if (out_ids)
    rc = rf_argmax(logits, rows, c.vocab, c.vocab_ld, out_ids, out_vals, 0, s.at(s.off_argmax), s.argmax_bytes, c.dtype, st);
  return rc;
}

extern "C" void rf_mixed_struct_sizes(int32_t* out) {
  out[0] = (int32_t)sizeof(RfMixedConfig); out[1] = (int32_t)sizeof(RfMixedLayer); out[2] = (int32_t)sizeof(RfMixedForward);
  out[3] = (int32_t)sizeof(RfRows); out[4] = (int32_t)sizeof(RfStreamNorm); out[5] = (int32_t)sizeof(RfLatentAttn);
  out[6] = (int32_t)sizeof(RfHgrn2); out[7] = (int32_t)sizeof(RfHeadLinear);
}
