// Vizotar model body behind the step executor (runner.cu): weights, per-layer paged key / value pools and recurrent state slots, the
// layer loop.
//
// The residual is `streams` fp32 rows per token.  One sublayer q (1: mixer, 2: feed-forward) of a layer over the N query rows of a step:
//   nvc_streams_norm          closes the previous sublayer (X_t <- sum_s mix[s, t] X_s + out_t y; y = its output, or the two outputs of
//                             a parallel mixer normed over the width and averaged) and opens this one (h = norm(sum_s in_s X_s))
//   parallel:
//     linear w_in             ONE fused projection of everything both mixers read from h, fp32 out:
//                             [q | k | v | memory q | k | v | gate | i | f]
//     nvc_qkv_prep_run        biases, short convolutions, norms over the whole query / key projection, rotary positions, k / v into this
//                             layer's paged pools;  nvc_short_conv_advance (portions only): the convolution state
//     nvc_attn_paged_wide     window and sink (long portions of 128-wide heads: nvc_prefill_attn_paged_window)
//     nvc_memory_scan         gates and the matrix memory, straight from the projection rows;  nvc_group_norm_gate: per-head norm,
//                             weight, sigmoid gate
//     linear o (left, its bias rides on the next nvc_streams_norm), linear o (right)
//   channel_delta:
//     linear w_in             [q | k | v | beta | a1 | g1], fp32 out;  the two low-rank parts in the storage format -> linear w_low: decays
//                             and gate in one product (block-diagonal weights)
//     nvc_delta_prep_run      short convolutions + silu, unit q / k, log decays per channel, beta;  nvc_delta_rule_scan;
//     nvc_head_gate_w         per-head root mean square, weight, sigmoid gate;  linear o
//   dense ff:  linear [gate; up] with the clamped gated unit in its epilogue -> linear down (fp32)
//   moe ff:    routed_experts.h: biased logits, softmax over the chosen
// A layer with `weights_of` runs another layer's weights with pools and state of its own.
//
// The inner sizes of the low-rank projections come from the checkpoint's shapes, so the fused projection of a channel_delta layer gets
// its final height when all tensors are there (finalize).  Feature dimensions that a dense matrix product sums over or produces are
// padded to multiples of 64 (zeros), so that the tcgen05 GEMMs take every such product of the bf16 mode; heads are not padded.
#include <cmath>
#include <cstring>
#include <string>
#include <vector>

#include "body_common.h"
#include "model_config.h"
#include "routed_experts.h"
#include "runner.h"

namespace {

constexpr float kGluAlpha = 1.702f;      // g * sigmoid(alpha g) of the dense gated unit
constexpr float kUnitEps = 1e-6f;        // inside the root of the delta rule's unit vectors
constexpr float kMemoryEps = 1e-6f;      // in the memory's denominator

inline int pad16(int v) { return (v + 15) / 16 * 16; }

struct VSublayerW {                     // a sublayer's norm and its place among the streams
  float *norm = nullptr, *in = nullptr, *out = nullptr, *mix = nullptr;
};

struct VLayerW {
  VSublayerW sub[2];
  void* w_in = nullptr;                 // [np, Wp]
  int np = 0;
  int q_off = 0, k_off = 0, v_off = 0;  // left half of "parallel", or the delta mixer
  // parallel
  int mq_off = 0, mk_off = 0, mv_off = 0, mg_off = 0, i_off = 0, f_off = 0;
  float *bias = nullptr, *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr, *o_bias = nullptr, *out_l = nullptr, *out_r = nullptr;
  float *mem_norm = nullptr, *i_bias = nullptr, *f_bias = nullptr;
  const float* rot = nullptr;
  void* w_o2 = nullptr;                 // [Wp, owp2]
  int owp2 = 0;
  // channel_delta
  int b_off = 0, low_off = 0;
  float *A_log = nullptr, *dt_bias = nullptr, *onorm = nullptr;
  int a_rank = 0, g_rank = 0, ap = 0, lowp = 0;     // ranks, a1's padded width, both padded widths
  int gl_off = 0, lnp = 0;              // first gate column, width of the low-rank product
  std::vector<float> a1, g1, a2, g2;    // host copies until finalize
  void* w_low = nullptr;                // [lnp, lowp]: decay rows read the a1 part, gate rows the g1 part
  // both
  float* conv_w = nullptr;              // tap-major [taps, channels of q | k | v]
  void* w_o = nullptr;                  // [Wp, owp]
  int owp = 0;
  // dense ff
  void *w_gu = nullptr, *w_down = nullptr;          // [2 ffp, Wp] (16 gate rows, 16 up rows, ...; without tcgen05: all gate rows, all up rows), [Wp, ffp]
  int ffp = 0;
  nvc_experts_weights moe;
};

struct VRunState {                      // what one layer keeps between steps
  void *k_cache = nullptr, *v_cache = nullptr;      // [slots, kv_heads * dim], [slots, kv_heads * vdim]
  float* conv_state = nullptr;                      // [state slots, taps - 1, channels]
  float *state = nullptr, *nm_state = nullptr;      // [state slots, heads, dim, vdim]; the memory's normaliser and maximum
};

struct VizotarBody : nvc_body_base {
  nvc_vizotar_config cfg;
  int Wp = 0, Vp = 0, ldx = 0;          // ldx: floats between two tokens' streams
  int state_slots = 0;
  nvc_experts experts{{"mlp.router.b", NVC_ROUTE_CHOSEN, 1, NVC_ACT_SILU_MUL, 0.f}};
  std::vector<VLayerW> L;
  std::vector<VRunState> R;
  void* embed = nullptr;
  float* fw = nullptr;
  // activations
  size_t T = 0;
  float *x0 = nullptr, *X = nullptr, *proj = nullptr, *mix = nullptr, *mix2 = nullptr, *ffo = nullptr;
  float *rq = nullptr, *rk = nullptr, *rv = nullptr, *ro = nullptr, *gb = nullptr, *lowf = nullptr, *gch = nullptr;
  void *h = nullptr, *q = nullptr, *ao = nullptr, *ao2 = nullptr, *low = nullptr, *gu = nullptr, *act = nullptr, *hn = nullptr;
  float* tap_host = nullptr;
  size_t tap_cap = 0;

  int vocab() const override { return cfg.vocab; }
  int logits_ld() const override { return Vp; }
  int layer_runs() const override { return (int)cfg.layers.size(); }
  int width() const override { return cfg.width; }
  int num_state_slots() const override { return state_slots; }
  int64_t cache_bytes_per_token() const override {
    int64_t b = 0;
    for (auto& ly : cfg.layers)
      if (ly.kind == nvc_vizotar_layer::Parallel) b += (int64_t)ly.attn.kv_heads * (ly.attn.dim + ly.attn.vdim) * (int64_t)esz;
    return b;
  }
  int set_residual_tap(float* host, size_t cap) override {
    tap_host = host;
    tap_cap = host ? cap : 0;
    return NVC_OK;
  }

  static int attn_channels(const nvc_window_attn_spec& a) { return a.heads * a.dim + a.kv_heads * (a.dim + a.vdim); }
  static int delta_channels(const nvc_delta_spec& d) { return 2 * d.kv_heads * d.dim + d.heads * d.vdim; }
  static int slices(int vdim) { return (vdim + 31) / 32; }

  int init(nvc_runner* r) {
    dt = r->dtype;
    esz = dt == NVC_DT_F32 ? 4 : 2;
    use_tc = dt == NVC_DT_BF16 && !(getenv("NVC_VIZOTAR_TC") && atoi(getenv("NVC_VIZOTAR_TC")) == 0);
    experts.use_tc = use_tc && !(getenv("NVC_VIZOTAR_MOE_TC") && atoi(getenv("NVC_VIZOTAR_MOE_TC")) == 0);
    use_flash = use_tc && !(getenv("NVC_VIZOTAR_FLASH") && atoi(getenv("NVC_VIZOTAR_FLASH")) == 0);
    Wp = pad64(cfg.width);
    Vp = pad64(cfg.vocab);
    ldx = cfg.streams * Wp;
    state_slots = r->opt.max_num_seqs;
    T = (size_t)std::max(r->opt.max_num_batched_tokens, r->opt.max_num_seqs);
    const size_t slots = (size_t)r->opt.num_kvcache_blocks * r->opt.kvcache_block_size;
    const int W = cfg.width, S = cfg.streams;
    int rc;
    L.resize(cfg.layers.size());
    R.resize(cfg.layers.size());
    size_t m_q = 0, m_ow = 0, m_ow2 = 0, m_ff = 0, m_dqk = 0, m_dv = 0, m_gb = 0, m_g = 0;
    int64_t wbytes = 0;
    for (size_t i = 0; i < cfg.layers.size(); ++i) {
      const auto& ly = cfg.layers[i];
      if (ly.weights_of >= 0) continue;
      VLayerW& w = L[i];
      const std::string p = "l" + std::to_string(i) + ".";
      const auto& f = ly.mlp;
      for (int k = 0; k < (f.kind == nvc_routed_mlp_spec::None ? 1 : 2); ++k) {
        const std::string hc = p + "hc" + std::to_string(k + 1) + ".";
        VSublayerW& s = w.sub[k];
        if ((rc = zalloc(r, &s.norm, W * 4)) || (rc = zalloc(r, &s.in, S * 4)) || (rc = zalloc(r, &s.out, S * 4)) || (rc = zalloc(r, &s.mix, S * S * 4)))
          return rc;
        want[p + "norm" + std::to_string(k + 1)] = false;
        for (const char* n : {"in", "out", "mix"}) want[hc + n] = false;
      }
      int ow = 0;
      if (ly.kind == nvc_vizotar_layer::Parallel) {
        const auto& a = ly.attn;
        const auto& d = ly.mem;
        const int qw = a.heads * a.dim, kw = a.kv_heads * a.dim, vw = a.kv_heads * a.vdim, inner = d.heads * d.vdim;
        NVC_REQUIRE(r->ctx, a.dim <= 512 && a.vdim <= 512 && d.dim <= 1024, NVC_ESHAPE, "attention heads above 512 or memory keys above 1024 numbers");
        w.q_off = 0; w.k_off = qw; w.v_off = qw + kw;
        w.mq_off = pad16(w.v_off + vw);
        w.mk_off = pad16(w.mq_off + d.heads * d.dim);
        w.mv_off = pad16(w.mk_off + d.heads * d.dim);
        w.mg_off = pad16(w.mv_off + inner);
        w.i_off = pad16(w.mg_off + inner);
        w.f_off = w.i_off + d.heads;
        w.np = pad64(w.f_off + d.heads);
        ow = a.heads * a.vdim;
        w.owp2 = pad64(inner);
        if ((rc = zalloc(r, &w.bias, (size_t)w.np * 4)) || (rc = zalloc(r, &w.q_norm, qw * 4)) || (rc = zalloc(r, &w.k_norm, kw * 4)) ||
            (rc = zalloc(r, &w.sink, a.heads * 4)) || (rc = zalloc(r, &w.o_bias, W * 4)) || (rc = zalloc(r, &w.out_l, W * 4)) ||
            (rc = zalloc(r, &w.out_r, W * 4)) || (rc = zalloc(r, &w.mem_norm, inner * 4)) || (rc = zalloc(r, &w.i_bias, d.heads * 4)) ||
            (rc = zalloc(r, &w.f_bias, d.heads * 4)) || (rc = zalloc(r, &w.conv_w, (size_t)a.taps * attn_channels(a) * 4)) ||
            (rc = zalloc(r, &w.w_in, (size_t)w.np * Wp * esz)) || (rc = zalloc(r, &w.w_o2, (size_t)Wp * w.owp2 * esz)))
          return rc;
        if ((rc = rotary_table(r, a.rot, &w.rot))) return rc;
        for (const char* n : {"q", "q.b", "q.conv", "q.norm", "k", "k.b", "k.conv", "k.norm", "v", "v.b", "v.conv", "sink", "o", "o.b", "out"})
          want[p + "mix.left." + n] = false;
        for (const char* n : {"q", "k", "v", "g", "o", "norm", "i", "i.b", "f", "f.b", "out"}) want[p + "mix.right." + n] = false;
        wbytes += (int64_t)esz * ((int64_t)(qw + kw + vw + 2 * d.heads * (d.dim + 1) + 2 * inner) * W + (int64_t)W * (ow + inner));
        m_q = std::max(m_q, (size_t)qw);
        m_ow2 = std::max(m_ow2, (size_t)w.owp2);
        m_dv = std::max(m_dv, (size_t)inner);
      } else {
        const auto& d = ly.delta;
        const int qk = d.kv_heads * d.dim, vw = d.heads * d.vdim;
        NVC_REQUIRE(r->ctx, d.dim <= 1024, NVC_ESHAPE, "delta-rule keys above 1024 numbers");
        w.q_off = 0; w.k_off = qk; w.v_off = 2 * qk; w.b_off = pad16(2 * qk + vw); w.low_off = pad16(w.b_off + d.heads);
        ow = vw;
        if ((rc = zalloc(r, &w.A_log, d.heads * 4)) || (rc = zalloc(r, &w.dt_bias, (size_t)d.heads * d.dim * 4)) || (rc = zalloc(r, &w.onorm, d.vdim * 4)) ||
            (rc = zalloc(r, &w.conv_w, (size_t)d.taps * delta_channels(d) * 4)) || (rc = zalloc(r, &w.w_in, (size_t)w.low_off * Wp * esz)))
          return rc;
        for (const char* n : {"q", "q.conv", "k", "k.conv", "v", "v.conv", "b", "A_log", "dt_bias", "norm", "a1", "a2", "g1", "g2", "o"})
          want[p + "mix." + n] = false;
        wbytes += (int64_t)esz * ((int64_t)(2 * qk + vw + d.heads) * W + (int64_t)W * vw);
        m_dqk = std::max(m_dqk, (size_t)qk);
        m_dv = std::max(m_dv, (size_t)vw);
        m_gb = std::max(m_gb, (size_t)2 * d.heads);
        m_g = std::max(m_g, (size_t)d.heads * d.dim);
      }
      w.owp = pad64(ow);
      if ((rc = zalloc(r, &w.w_o, (size_t)Wp * w.owp * esz))) return rc;
      m_ow = std::max(m_ow, (size_t)w.owp);
      if (f.kind == nvc_routed_mlp_spec::Dense) {
        w.ffp = pad64(f.ff);
        if ((rc = zalloc(r, &w.w_gu, (size_t)2 * w.ffp * Wp * esz)) || (rc = zalloc(r, &w.w_down, (size_t)Wp * w.ffp * esz))) return rc;
        for (const char* n : {"gate", "up", "down"}) want[p + "mlp." + n] = false;
        wbytes += (int64_t)esz * 3 * f.ff * W;
        m_ff = std::max(m_ff, (size_t)w.ffp);
      } else if (f.kind == nvc_routed_mlp_spec::Moe) {
        if ((rc = experts.init(*this, r, f, p, W, T, w.moe, &wbytes))) return rc;
      }
    }
    // pools and state of every layer, also of those that borrow their weights
    for (size_t i = 0; i < cfg.layers.size(); ++i) {
      const auto& ly = cfg.layers[i];
      VRunState& s = R[i];
      if (ly.kind == nvc_vizotar_layer::Parallel) {
        const auto& a = ly.attn;
        const auto& d = ly.mem;
        if ((rc = zalloc(r, &s.k_cache, slots * a.kv_heads * a.dim * esz)) || (rc = zalloc(r, &s.v_cache, slots * a.kv_heads * a.vdim * esz)) ||
            (rc = zalloc(r, &s.conv_state, (size_t)state_slots * std::max(a.taps - 1, 1) * attn_channels(a) * 4)) ||
            (rc = zalloc(r, &s.state, (size_t)state_slots * d.heads * d.dim * d.vdim * 4)) ||
            (rc = zalloc(r, &s.nm_state, (size_t)state_slots * d.heads * slices(d.vdim) * (d.dim + 1) * 4)))
          return rc;
      } else {
        const auto& d = ly.delta;
        if ((rc = zalloc(r, &s.conv_state, (size_t)state_slots * std::max(d.taps - 1, 1) * delta_channels(d) * 4)) ||
            (rc = zalloc(r, &s.state, (size_t)state_slots * d.heads * d.dim * d.vdim * 4)))
          return rc;
      }
    }
    if ((rc = zalloc(r, &embed, (size_t)Vp * Wp * esz)) || (rc = zalloc(r, &fw, W * 4))) return rc;
    want["embed"] = false;
    want["final.norm"] = false;
    r->weight_bytes = wbytes + (int64_t)esz * cfg.vocab * W;      // the low-rank projections join in finalize
    // activations (zeroed once: padding columns are never written)
    if ((rc = zalloc(r, &x0, T * Wp * 4)) || (rc = zalloc(r, &X, T * ldx * 4)) || (rc = zalloc(r, &mix, T * Wp * 4)) ||
        (rc = zalloc(r, &ffo, T * Wp * 4)) || (rc = zalloc(r, &h, T * Wp * esz)) || (rc = zalloc(r, &ao, T * m_ow * esz)) ||
        (rc = zalloc(r, &hn, (size_t)r->max_logit_rows * Wp * esz)) || (rc = zalloc(r, &ro, T * m_dv * 4)))
      return rc;
    if (m_q && ((rc = zalloc(r, &q, T * m_q * esz)) || (rc = zalloc(r, &ao2, T * m_ow2 * esz)) || (rc = zalloc(r, &mix2, T * Wp * 4)))) return rc;
    if (m_dqk && ((rc = zalloc(r, &rq, T * m_dqk * 4)) || (rc = zalloc(r, &rk, T * m_dqk * 4)) || (rc = zalloc(r, &rv, T * m_dv * 4)) ||
                  (rc = zalloc(r, &gb, T * m_gb * 4)) || (rc = zalloc(r, &gch, T * m_g * 4))))
      return rc;
    if (m_ff && ((!use_tc && (rc = zalloc(r, &gu, T * 2 * m_ff * esz))) || (rc = zalloc(r, &act, T * m_ff * esz)))) return rc;
    return experts.alloc(*this, r, Wp, T);
  }

  int load_tensor(nvc_runner* r, const char* cname, const void* data, int st_dtype, const int64_t* shape, int ndim) override {
    nvc_ctx* ctx = r->ctx;
    const std::string name(cname);
    auto it = want.find(name);
    if (it == want.end()) return NVC_OK;    // not a tensor of this configuration: ignored
    size_t n = 1;
    for (int i = 0; i < ndim; ++i) n *= (size_t)shape[i];
    std::vector<float> v;
    NVC_REQUIRE(ctx, tensor_to_f32(data, st_dtype, n, v), NVC_EINVAL, "unsupported dtype for " + name);
    const int64_t d0 = ndim > 0 ? shape[0] : 1, d1 = ndim > 1 ? shape[1] : 1;
    auto shape_is = [&](int64_t a, int64_t b) { return (ndim <= 2) && d0 == a && d1 == b && (ndim == 2 || b == 1); };
    auto bad = [&]() {
      nvc_set_error(ctx, "unexpected shape for " + name);
      return NVC_ESHAPE;
    };
    const int W = cfg.width, S = cfg.streams;
    auto vec = [&](float* dst, size_t len) { return n == len ? put_f32(r, dst, v.data(), len) : bad(); };
    int rc = NVC_OK;
    if (name == "embed") { if (!shape_is(cfg.vocab, W)) return bad(); rc = put_matrix(r, embed, Wp, 0, 0, v.data(), cfg.vocab, W, W, 1); }
    else if (name == "final.norm") rc = vec(fw, W);
    else {
      const size_t dot = name.find('.');
      const int li = atoi(name.substr(1, dot - 1).c_str());
      const std::string sub = name.substr(dot + 1);
      const auto& ly = cfg.layers[li];
      const auto& f = ly.mlp;
      VLayerW& w = L[li];
      auto in_rows = [&](int off, int rows) { return shape_is(rows, W) ? put_matrix(r, w.w_in, Wp, off, 0, v.data(), rows, W, W, 1) : bad(); };
      auto out_matrix = [&](void* dst, int ldo, int cols) { return shape_is(W, cols) ? put_matrix(r, dst, ldo, 0, 0, v.data(), W, cols, cols, 1) : bad(); };
      // [channels, taps] of the checkpoint -> tap-major [taps, all channels] (q, k, v side by side): a warp's lanes read neighbours
      auto conv = [&](int taps, int ch0, int rows, int C) -> int {
        if (!shape_is(rows, taps)) return bad();
        std::vector<float> col(rows);
        int e = NVC_OK;
        for (int i = 0; i < taps && e == NVC_OK; ++i) {
          for (int c = 0; c < rows; ++c) col[c] = v[(size_t)c * taps + i];
          e = put_f32(r, w.conv_w + (size_t)i * C + ch0, col.data(), rows);
        }
        return e;
      };
      bool taken = false;
      rc = experts.load(*this, r, f, W, w.moe, sub, v, d0, d1, bad, &taken);
      if (taken) {
        it->second = rc == NVC_OK;
        return rc;
      }
      if (sub.rfind("hc", 0) == 0 || sub.rfind("norm", 0) == 0) {
        VSublayerW& s = w.sub[sub.find('2') == std::string::npos ? 0 : 1];
        if (sub.rfind("norm", 0) == 0) rc = vec(s.norm, W);
        else if (sub.substr(4) == "in") rc = vec(s.in, S);
        else if (sub.substr(4) == "out") rc = vec(s.out, S);
        else rc = shape_is(S, S) ? put_f32(r, s.mix, v.data(), n) : bad();
      } else if (ly.kind == nvc_vizotar_layer::Parallel && sub.rfind("mix.left.", 0) == 0) {
        const auto& a = ly.attn;
        const std::string t = sub.substr(9);
        const int qw = a.heads * a.dim, kw = a.kv_heads * a.dim, vw = a.kv_heads * a.vdim, C = attn_channels(a);
        if (t == "q") rc = in_rows(w.q_off, qw);
        else if (t == "k") rc = in_rows(w.k_off, kw);
        else if (t == "v") rc = in_rows(w.v_off, vw);
        else if (t == "q.b") rc = vec(w.bias + w.q_off, qw);
        else if (t == "k.b") rc = vec(w.bias + w.k_off, kw);
        else if (t == "v.b") rc = vec(w.bias + w.v_off, vw);
        else if (t == "q.conv") rc = conv(a.taps, 0, qw, C);
        else if (t == "k.conv") rc = conv(a.taps, qw, kw, C);
        else if (t == "v.conv") rc = conv(a.taps, qw + kw, vw, C);
        else if (t == "q.norm") rc = vec(w.q_norm, qw);
        else if (t == "k.norm") rc = vec(w.k_norm, kw);
        else if (t == "sink") rc = vec(w.sink, a.heads);
        else if (t == "o") rc = out_matrix(w.w_o, w.owp, a.heads * a.vdim);
        else if (t == "o.b") rc = vec(w.o_bias, W);
        else if (t == "out") rc = vec(w.out_l, W);
      } else if (ly.kind == nvc_vizotar_layer::Parallel && sub.rfind("mix.right.", 0) == 0) {
        const auto& d = ly.mem;
        const std::string t = sub.substr(10);
        const int inner = d.heads * d.vdim;
        if (t == "q") rc = in_rows(w.mq_off, d.heads * d.dim);
        else if (t == "k") rc = in_rows(w.mk_off, d.heads * d.dim);
        else if (t == "v") rc = in_rows(w.mv_off, inner);
        else if (t == "g") rc = in_rows(w.mg_off, inner);
        else if (t == "i") rc = in_rows(w.i_off, d.heads);
        else if (t == "f") rc = in_rows(w.f_off, d.heads);
        else if (t == "i.b") rc = vec(w.i_bias, d.heads);
        else if (t == "f.b") rc = vec(w.f_bias, d.heads);
        else if (t == "norm") rc = vec(w.mem_norm, inner);
        else if (t == "o") rc = out_matrix(w.w_o2, w.owp2, inner);
        else if (t == "out") rc = vec(w.out_r, W);
      } else if (ly.kind == nvc_vizotar_layer::ChannelDelta && sub.rfind("mix.", 0) == 0) {
        const auto& d = ly.delta;
        const std::string t = sub.substr(4);
        const int qk = d.kv_heads * d.dim, vw = d.heads * d.vdim, C = delta_channels(d);
        if (t == "q") rc = in_rows(w.q_off, qk);
        else if (t == "k") rc = in_rows(w.k_off, qk);
        else if (t == "v") rc = in_rows(w.v_off, vw);
        else if (t == "b") rc = in_rows(w.b_off, d.heads);
        else if (t == "q.conv") rc = conv(d.taps, 0, qk, C);
        else if (t == "k.conv") rc = conv(d.taps, qk, qk, C);
        else if (t == "v.conv") rc = conv(d.taps, 2 * qk, vw, C);
        else if (t == "A_log") rc = vec(w.A_log, d.heads);
        else if (t == "dt_bias") rc = vec(w.dt_bias, (size_t)d.heads * d.dim);
        else if (t == "norm") rc = vec(w.onorm, d.vdim);
        else if (t == "o") rc = out_matrix(w.w_o, w.owp, vw);
        else if (t == "a1" || t == "g1") {
          if (ndim != 2 || d1 != W) return bad();
          (t == "a1" ? w.a_rank : w.g_rank) = (int)d0;
          (t == "a1" ? w.a1 : w.g1) = std::move(v);
        } else if (t == "a2" || t == "g2") {
          if (ndim != 2 || d0 != (t == "a2" ? d.heads * d.dim : vw)) return bad();
          (t == "a2" ? w.a2 : w.g2) = std::move(v);
        }
      } else if (f.kind == nvc_routed_mlp_spec::Dense) {
        if (sub == "mlp.down") rc = out_matrix(w.w_down, w.ffp, f.ff);
        else if (!shape_is(f.ff, W)) return bad();
        else if (!use_tc) rc = put_matrix(r, w.w_gu, Wp, sub == "mlp.up" ? w.ffp : 0, 0, v.data(), f.ff, W, W, 1);
        else
          for (int j = 0; j < f.ff && rc == NVC_OK; j += 16)
            rc = put_matrix(r, w.w_gu, Wp, 2 * j + (sub == "mlp.up" ? 16 : 0), 0, v.data() + (size_t)j * W, std::min(16, f.ff - j), W, W, 1);
      }
    }
    if (rc == NVC_OK) it->second = true;
    return rc;
  }

  // with every tensor there the ranks of the low-rank projections are known: the fused projections of the delta layers get their last
  // rows, and the buffers that depend on the ranks their sizes
  int finalize(nvc_runner* r) override {
    int rc = require_all_tensors(r);
    if (rc) return rc;
    if (proj) return NVC_OK;             // called before
    const int W = cfg.width;
    size_t m_np = 0, m_low = 0, m_lnp = 0;
    for (size_t i = 0; i < L.size(); ++i) {
      const auto& ly = cfg.layers[i];
      if (ly.weights_of >= 0) continue;
      VLayerW& w = L[i];
      if (ly.kind == nvc_vizotar_layer::ChannelDelta) {
        const auto& d = ly.delta;
        const int gw = d.heads * d.dim, vw = d.heads * d.vdim;
        NVC_REQUIRE(r->ctx, w.a_rank > 0 && w.g_rank > 0 && w.a2.size() == (size_t)gw * w.a_rank && w.g2.size() == (size_t)vw * w.g_rank, NVC_ESHAPE,
                    "l" + std::to_string(i) + ": the halves of a low-rank projection do not fit");
        w.ap = pad64(w.a_rank);
        w.lowp = w.ap + pad64(w.g_rank);
        w.gl_off = pad16(gw);
        w.lnp = pad64(w.gl_off + vw);
        w.np = pad64(w.low_off + w.lowp);
        void* grown = nullptr;
        if ((rc = zalloc(r, &grown, (size_t)w.np * Wp * esz)) || (rc = zalloc(r, &w.w_low, (size_t)w.lnp * w.lowp * esz))) return rc;
        NVC_CUDA_CHECK(r->ctx, cudaMemcpy(grown, w.w_in, (size_t)w.low_off * Wp * esz, cudaMemcpyDeviceToDevice));
        r->allocs.erase(std::remove(r->allocs.begin(), r->allocs.end(), w.w_in), r->allocs.end());
        NVC_CUDA_CHECK(r->ctx, cudaFree(w.w_in));
        w.w_in = grown;
        if ((rc = put_matrix(r, w.w_in, Wp, w.low_off, 0, w.a1.data(), w.a_rank, W, W, 1)) ||
            (rc = put_matrix(r, w.w_in, Wp, w.low_off + w.ap, 0, w.g1.data(), w.g_rank, W, W, 1)) ||
            (rc = put_matrix(r, w.w_low, w.lowp, 0, 0, w.a2.data(), gw, w.a_rank, w.a_rank, 1)) ||
            (rc = put_matrix(r, w.w_low, w.lowp, w.gl_off, w.ap, w.g2.data(), vw, w.g_rank, w.g_rank, 1)))
          return rc;
        for (auto* t : {&w.a1, &w.g1, &w.a2, &w.g2}) std::vector<float>().swap(*t);
        r->weight_bytes += (int64_t)esz * ((int64_t)(w.a_rank + w.g_rank) * W + (int64_t)gw * w.a_rank + (int64_t)vw * w.g_rank);
        m_low = std::max(m_low, (size_t)w.lowp);
        m_lnp = std::max(m_lnp, (size_t)w.lnp);
      }
      m_np = std::max(m_np, (size_t)w.np);
    }
    if ((rc = zalloc(r, &proj, T * m_np * 4))) return rc;
    if (m_low && ((rc = zalloc(r, &low, T * m_low * esz)) || (rc = zalloc(r, &lowf, T * m_lnp * 4)))) return rc;
    return NVC_OK;
  }

  // left half of a parallel mixer into ao[:, :heads * vdim]
  int window_attention(nvc_runner* r, const nvc_step_shape& s, const nvc_window_attn_spec& a, const VLayerW& w, const VRunState& rs) {
    nvc_ctx* ctx = r->ctx;
    void* st = r->stream;
    nvc_short_conv cv{a.taps, w.conv_w, rs.conv_state, r->d_state_slots, s.decode ? nullptr : r->d_cu, s.B};
    nvc_qkv_prep p{};
    p.in = proj; p.ldi = w.np;
    p.bias = w.bias;
    p.q_off = w.q_off; p.k_off = w.k_off; p.v_off = w.v_off;
    p.q_heads = a.heads; p.kv_heads = a.kv_heads; p.dim = a.dim; p.vdim = a.vdim;
    p.q_norm = w.q_norm; p.k_norm = w.k_norm; p.eps = cfg.eps; p.wide_norm = 1;
    p.rot_dims = a.rot.dims; p.rot_half = 1; p.rot_table = w.rot; p.positions = r->d_pos;
    p.k_scale = 1.f; p.v_scale = 1.f;
    p.blend = NVC_BLEND_NONE;
    p.q_out = q; p.ldq = a.heads * a.dim;
    p.k_out = rs.k_cache; p.v_out = rs.v_cache; p.ldk = a.kv_heads * a.dim; p.ldv = a.kv_heads * a.vdim;
    p.slot_mapping = r->d_slots;
    p.q_dtype = dt; p.kv_dtype = dt;
    p.conv = &cv;
    int rc = nvc_qkv_prep_run(ctx, &p, s.N, st);
    if (rc) return rc;
    if (!s.decode && (rc = nvc_short_conv_advance(ctx, &cv, proj, w.np, w.q_off, w.bias + w.q_off, attn_channels(a), r->d_pos, st))) return rc;
    mark(r, "qkv_prep");
    nvc_attn_spec sp{};
    sp.heads = a.heads; sp.kv_heads = a.kv_heads; sp.dim = a.dim; sp.vdim = a.vdim;
    sp.scale = a.scale;
    sp.window = a.window;
    sp.sink = w.sink;
    sp.out_scale = 1.f;
    const int bs = r->opt.kvcache_block_size, cap = r->max_blocks_cap;
    if (a.dim == 128 && a.vdim == 128 && a.scale > 0.f && flash_step(r, s)) {
      // portions with 128-wide keys and values take the tcgen05 kernel; the one-token sequences of a mixed step come first in the batch and
      // keep the decode path of the wide kernel
      const int nd = s.num_decode;
      if (nd > 0 && (rc = nvc_attn_paged_wide(ctx, q, p.ldq, rs.k_cache, p.ldk, rs.v_cache, p.ldv, r->d_bt, cap, r->d_ctx, nullptr, nd, nd, 1, bs, &sp, ao,
                                              w.owp, dt, st)))
        return rc;
      rc = nvc_prefill_attn_paged_window(ctx, reinterpret_cast<const nvc_bf16*>(q) + (size_t)nd * p.ldq, p.ldq, reinterpret_cast<const nvc_bf16*>(rs.k_cache),
                                         reinterpret_cast<const nvc_bf16*>(rs.v_cache), r->d_bt + (size_t)nd * cap, cap, r->d_ctx + nd,
                                         nd ? r->d_cu2 : r->d_cu, s.B - nd, s.N - nd, s.max_chunk, a.heads, a.kv_heads, 128, bs,
                                         r->opt.num_kvcache_blocks, a.scale, a.window, w.sink, reinterpret_cast<nvc_bf16*>(ao) + (size_t)nd * w.owp, w.owp, st);
    } else {
      rc = nvc_attn_paged_wide(ctx, q, p.ldq, rs.k_cache, p.ldk, rs.v_cache, p.ldv, r->d_bt, cap, r->d_ctx, s.decode ? nullptr : r->d_cu, s.B, s.N,
                               s.decode ? 1 : s.max_seqlen, bs, &sp, ao, w.owp, dt, st);
    }
    mark(r, "attention");
    return rc;
  }

  // right half of a parallel mixer into ao2[:, :heads * vdim]
  int memory_mixer(nvc_runner* r, const nvc_step_shape& s, const nvc_memory_spec& d, const VLayerW& w, const VRunState& rs) {
    nvc_ctx* ctx = r->ctx;
    void* st = r->stream;
    const int inner = d.heads * d.vdim;
    nvc_memory_scan_args m{};
    m.q = proj + w.mq_off; m.k = proj + w.mk_off; m.v = proj + w.mv_off;
    m.ldq = m.ldk = m.ldv = w.np;
    m.q_scale = 1.0f / sqrtf((float)d.dim);
    m.i_in = proj + w.i_off; m.f_in = proj + w.f_off; m.ldg = w.np;
    m.i_bias = w.i_bias; m.f_bias = w.f_bias; m.cap = d.gate_cap; m.den_eps = kMemoryEps;
    m.o = ro; m.ldo = inner;
    m.state = rs.state; m.nm_state = rs.nm_state; m.state_slots = r->d_state_slots; m.cu_seqlens = s.decode ? nullptr : r->d_cu; m.positions = r->d_pos;
    m.heads = d.heads; m.dim = d.dim; m.vdim = d.vdim;
    int rc = nvc_memory_scan(ctx, &m, s.B, s.decode ? 1 : s.max_seqlen, st);
    if (rc) return rc;
    mark(r, "memory_scan");
    rc = nvc_group_norm_gate(ctx, ro, inner, proj + w.mg_off, w.np, w.mem_norm, ao2, w.owp2, dt, d.heads, d.vdim, 0, cfg.eps, NVC_GATE_SIGMOID, s.N, st);
    mark(r, "memory_norm_gate");
    return rc;
  }

  int delta_mixer(nvc_runner* r, const nvc_step_shape& s, const nvc_delta_spec& d, const VLayerW& w, const VRunState& rs) {
    nvc_ctx* ctx = r->ctx;
    void* st = r->stream;
    // the inner numbers of both low-rank projections in the storage format, then decays and gate in one product
    int rc = nvc_rms_norm_blend(ctx, proj + w.low_off, nullptr, nullptr, nullptr, 0.f, nullptr, nullptr, 0.f, nullptr, w.np, nullptr, low, dt, w.lowp,
                                cfg.eps, nullptr, s.N, w.lowp, st);
    if (rc) return rc;
    mark(r, "low_rank_cast");
    if ((rc = linear(r, low, w.lowp, w.w_low, lowf, w.lnp, NVC_DT_F32, s.N, w.lnp, w.lowp))) return rc;
    mark(r, "gemm_low_rank");
    nvc_delta_prep p{};
    p.in = proj; p.ldi = w.np;
    p.q_off = w.q_off; p.k_off = w.k_off; p.v_off = w.v_off; p.b_off = w.b_off;
    p.heads = d.heads; p.kv_heads = d.kv_heads; p.dim = d.dim; p.vdim = d.vdim; p.taps = d.taps;
    p.conv_w = w.conv_w; p.conv_state = rs.conv_state;
    p.state_slots = r->d_state_slots; p.cu_seqlens = s.decode ? nullptr : r->d_cu; p.positions = r->d_pos;
    p.A_log = w.A_log; p.dt_bias = w.dt_bias;
    p.unit_eps = kUnitEps; p.q_scale = 1.0f / sqrtf((float)d.dim);
    p.q_out = rq; p.k_out = rk; p.v_out = rv; p.ldq = p.ldk = d.kv_heads * d.dim; p.ldv = d.heads * d.vdim;
    p.gb_out = gb;
    p.B = s.B;
    p.channel_a = lowf; p.ldca = w.lnp; p.channel_g = gch;
    if ((rc = nvc_delta_prep_run(ctx, &p, s.N, s.decode ? 1 : s.max_seqlen, st))) return rc;
    mark(r, "delta_prep");
    if ((rc = nvc_delta_rule_scan(ctx, &p, ro, p.ldv, rs.state, s.decode ? 1 : s.max_seqlen, st))) return rc;
    mark(r, "delta_scan");
    rc = nvc_head_gate_w(ctx, ro, p.ldv, lowf + w.gl_off, w.lnp, w.onorm, ao, w.owp, dt, d.heads, d.vdim, 1, cfg.eps, NVC_GATE_SIGMOID, 1.f, s.N, st);
    mark(r, "head_gate");
    return rc;
  }

  // a sublayer's output that has not reached the streams yet, and the weights that take it there
  struct Pending {
    const VSublayerW* sub = nullptr;
    const float *y0 = nullptr, *b0 = nullptr, *w0 = nullptr, *y1 = nullptr, *w1 = nullptr;
    float c0 = 1.f, c1 = 1.f;
  };
  bool in_x0 = true;                    // every stream is still the embedding row
  // closes pd (if any) on the streams, then: opens `next` (h = norm of what it reads), or sums the streams into out (norm: weight or NULL)
  int land(nvc_runner* r, Pending& pd, const VSublayerW* next, const float* norm, void* out, int out_dt, const int32_t* rows, int n) {
    nvc_streams_args a{};
    a.x_in = in_x0 ? x0 : X;
    a.ldx_in = in_x0 ? Wp : ldx;
    a.sx_in = in_x0 ? 0 : Wp;
    a.streams = cfg.streams;
    const bool last = !next && norm;     // the head reads the sum; nobody reads the streams again
    if (pd.sub && !last) {
      a.x_out = X; a.ldx_out = ldx; a.sx_out = Wp;
      in_x0 = false;
    }
    if (pd.sub) {
      a.y0 = pd.y0; a.b0 = pd.b0; a.w0 = pd.w0; a.c0 = pd.c0;
      a.y1 = pd.y1; a.w1 = pd.w1; a.c1 = pd.c1;
      a.ldy = Wp;
      a.mix = pd.sub->mix; a.out_w = pd.sub->out;
    }
    a.in_w = next ? next->in : nullptr;
    a.norm_w = next ? next->norm : norm;
    a.ldo = Wp; a.eps = cfg.eps; a.rows = rows;
    pd = Pending();
    return nvc_streams_norm(r->ctx, &a, next ? h : out, next ? dt : out_dt, n, cfg.width, r->stream);
  }

  int forward(nvc_runner* r, const nvc_step_shape& s) override {
    nvc_ctx* ctx = r->ctx;
    void* st = r->stream;
    const int N = s.N, W = cfg.width;
    cudaStreamCaptureStatus cap = cudaStreamCaptureStatusNone;
    cudaStreamIsCapturing(r->stream, &cap);
    prof_on = prof_armed && cap == cudaStreamCaptureStatusNone;
    if (prof_on) prof_armed = false;
    mark(r, "start");
    int rc = nvc_embed_gather_f32(ctx, r->d_ids, embed, dt, Wp, x0, Wp, N, W, st);
    if (rc) return rc;
    mark(r, "embed");
    Pending pd;
    in_x0 = true;
    for (size_t i = 0; i < cfg.layers.size(); ++i) {
      const auto& ly = cfg.layers[i];
      const VLayerW& w = L[cfg.owner((int)i)];
      const VRunState& rs = R[i];
      // ---- mixer
      if ((rc = land(r, pd, &w.sub[0], nullptr, nullptr, dt, nullptr, N))) return rc;
      mark(r, "streams_norm");
      if ((rc = linear(r, h, Wp, w.w_in, proj, w.np, NVC_DT_F32, N, w.np, Wp))) return rc;
      mark(r, "gemm_in");
      pd.sub = &w.sub[0];
      pd.y0 = mix;
      if (ly.kind == nvc_vizotar_layer::Parallel) {
        if ((rc = window_attention(r, s, ly.attn, w, rs))) return rc;
        if ((rc = memory_mixer(r, s, ly.mem, w, rs))) return rc;
        if ((rc = linear(r, ao, w.owp, w.w_o, mix, Wp, NVC_DT_F32, N, Wp, w.owp))) return rc;
        if ((rc = linear(r, ao2, w.owp2, w.w_o2, mix2, Wp, NVC_DT_F32, N, Wp, w.owp2))) return rc;
        pd.b0 = w.o_bias; pd.w0 = w.out_l; pd.c0 = 0.5f;
        pd.y1 = mix2; pd.w1 = w.out_r; pd.c1 = 0.5f;
      } else {
        if ((rc = delta_mixer(r, s, ly.delta, w, rs))) return rc;
        if ((rc = linear(r, ao, w.owp, w.w_o, mix, Wp, NVC_DT_F32, N, Wp, w.owp))) return rc;
      }
      mark(r, "gemm_o");
      // ---- feed-forward
      const auto& f = ly.mlp;
      if (f.kind != nvc_routed_mlp_spec::None) {
        if ((rc = land(r, pd, &w.sub[1], nullptr, nullptr, dt, nullptr, N))) return rc;
        mark(r, "streams_norm");
        if (f.kind == nvc_routed_mlp_spec::Dense) {
          if (use_tc) {        // the gated unit in the epilogue of the product
            if ((rc = nvc_gemm_bf16_glu_clamp_mul(ctx, reinterpret_cast<const nvc_bf16*>(h), Wp, reinterpret_cast<const nvc_bf16*>(w.w_gu),
                                                  reinterpret_cast<nvc_bf16*>(act), w.ffp, N, w.ffp, Wp, f.limit, st)))
              return rc;
            mark(r, "gemm_gate_up");
          } else {
            if ((rc = linear(r, h, Wp, w.w_gu, gu, 2 * w.ffp, dt, N, 2 * w.ffp, Wp))) return rc;
            mark(r, "gemm_gate_up");
            if ((rc = nvc_act_mul_p(ctx, gu, 2 * w.ffp, act, w.ffp, dt, N, f.ff, w.ffp, NVC_ACT_GLU_CLAMP, f.limit, kGluAlpha, st))) return rc;
            mark(r, "glu");
          }
          if ((rc = linear(r, act, w.ffp, w.w_down, ffo, Wp, NVC_DT_F32, N, Wp, w.ffp))) return rc;
          mark(r, "gemm_down");
        } else if ((rc = experts.run(*this, r, f, w.moe, h, ffo, N, W))) {
          return rc;
        }
        pd.sub = &w.sub[1];
        pd.y0 = ffo;
      }
      if (tap_host) {
        // debug: bring this layer's output to the streams and copy their sum out (through the buffer that the pending output does not use)
        float* sum = pd.y0 == mix ? ffo : mix;
        if ((rc = land(r, pd, nullptr, nullptr, sum, NVC_DT_F32, nullptr, N))) return rc;
        if ((rc = copy_tap(r, sum, Wp, tap_host, tap_cap, (int)i, N, W))) return rc;
      }
    }
    tap_host = nullptr;      // one step only
    // ---- head: the last update and the final norm of the wanted rows, logits against the embedding table
    if ((rc = land(r, pd, nullptr, fw, hn, dt, s.decode ? nullptr : r->d_last_rows, s.rows))) return rc;
    mark(r, "final_norm");
    rc = linear(r, hn, Wp, embed, r->logits, Vp, NVC_DT_F32, s.rows, Vp, Wp);
    mark(r, "lm_head");
    finish_profile(r);
    return rc;
  }
};

}  // namespace

nvc_model_body* nvc_make_vizotar_body(nvc_runner* r, const nvc_vizotar_config& cfg, int* status) {
  VizotarBody* b = new VizotarBody();
  b->cfg = cfg;
  *status = b->init(r);
  return b;
}
