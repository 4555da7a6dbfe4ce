// Fefozen model body behind the step executor (runner.cu): weights, paged latent pools, recurrent state slots, the layer loop.
//
// One layer over the N query rows of a step (x <- x + n1b(mixer(n1(x))); x <- x + n2b(ff(n2(x))); norm weights stored around zero):
//   nvc_rms_norm_sandwich     x += norm-behind(previous sublayer's output); h = norm-in-front(x): one pass over the row
//   latent attention:
//     linear w_in             ONE fused projection of everything the mixer reads from h, fp32 out: [dq | dkv | gate]
//     latent_run              (latent_mixer.h) latents, absorbed queries, attention over shared rows, value up-projection, gate
//     linear o
//   delta:
//     linear w_in             [q | k | v | beta | a | gate], fp32 out
//     nvc_delta_prep_run      short convolutions + silu, unit q / k, decay and beta;  nvc_delta_rule_scan: the recurrence over the
//                             state slots of the step's sequences (and the convolution state);  nvc_head_gate_w: per-head root mean
//                             square, weight, silu gate;  linear o
//   dense ff:  linear up with the tanh-gelu in its epilogue -> linear down (fp32)
//   moe ff:    router product (fp32) -> softmax scores, biased top-k -> sort -> grouped [gate; up] -> clamped gated unit ->
//              grouped down (fp32) -> combine (identity experts add the token's own h)
// The residual sum itself happens in the NEXT nvc_rms_norm_sandwich (or the final one), in fp32.
//
// Feature dimensions that a dense matrix product sums over or produces are padded to multiples of 64 in the weight and activation
// buffers (zeros), so that the tcgen05 GEMMs (K % 64, N % 16) take every such product of the bf16 mode; heads are not padded.
#include <cmath>
#include <cstring>
#include <map>
#include <string>
#include <vector>

#include "latent_mixer.h"
#include "routed_experts.h"
#include "runner.h"

namespace {

constexpr float kGluAlpha = 1.702f;      // g * sigmoid(alpha g) of the experts' gated unit
constexpr float kUnitEps = 1e-6f;        // inside the root of the delta rule's unit vectors

struct FLayerW {
  float *n1 = nullptr, *n1b = nullptr, *n2 = nullptr, *n2b = nullptr;
  void* w_in = nullptr;                 // [np, Wp]
  int np = 0;
  int g_off = 0;
  nvc_latent_weights lat;
  // delta
  int q_off = 0, k_off = 0, v_off = 0, b_off = 0, a_off = 0;
  float *conv_w = nullptr, *conv_state = nullptr, *A_log = nullptr, *dt_bias = nullptr, *onorm = nullptr, *state = nullptr;
  // both
  void* w_o = nullptr;                  // [Wp, owp]
  int owp = 0;
  // dense ff
  void *w_up = nullptr, *w_down = nullptr;
  int ffp = 0;
  nvc_experts_weights moe;
};

struct FefozenBody : nvc_latent_body {
  nvc_fefozen_config cfg;
  int Wp = 0, Vp = 0;
  int state_slots = 0;
  nvc_experts experts{{"mlp.correction", NVC_ROUTE_SOFTMAX, 0, NVC_ACT_GLU_CLAMP, kGluAlpha}};
  std::vector<FLayerW> L;
  void* embed = nullptr;
  float* fw = nullptr;
  // activations
  float *x0 = nullptr, *res = nullptr, *proj = nullptr, *mix = nullptr, *ffo = nullptr;
  float *rq = nullptr, *rk = nullptr, *rv = nullptr, *ro = nullptr, *gb = nullptr;
  void *h = nullptr, *ao = nullptr, *act = nullptr, *hn = nullptr;
  float* tap_host = nullptr;
  size_t tap_cap = 0;

  int vocab() const override { return cfg.vocab; }
  int logits_ld() const override { return Vp; }
  int layer_runs() const override { return (int)cfg.layers.size(); }
  int width() const override { return cfg.width; }
  int num_state_slots() const override { return state_slots; }
  int64_t cache_bytes_per_token() const override {
    int64_t b = 0;
    for (size_t i = 0; i < cfg.layers.size(); ++i)
      if (cfg.layers[i].kind == nvc_fefozen_layer::Latent && cfg.layers[i].lat.kv_from < 0) b += (int64_t)L[i].lat.ldpool * (int64_t)esz;
    return b;
  }
  int set_residual_tap(float* host, size_t cap) override {
    tap_host = host;
    tap_cap = host ? cap : 0;
    return NVC_OK;
  }

  int init(nvc_runner* r) {
    nvc_ctx* ctx = r->ctx;
    dt = r->dtype;
    esz = dt == NVC_DT_F32 ? 4 : 2;
    use_tc = dt == NVC_DT_BF16 && !(getenv("NVC_FEFOZEN_TC") && atoi(getenv("NVC_FEFOZEN_TC")) == 0);
    use_flash = use_tc && !(getenv("NVC_FEFOZEN_FLASH") && atoi(getenv("NVC_FEFOZEN_FLASH")) == 0);
    experts.use_tc = use_tc && !(getenv("NVC_FEFOZEN_MOE_TC") && atoi(getenv("NVC_FEFOZEN_MOE_TC")) == 0);
    Wp = pad64(cfg.width);
    Vp = pad64(cfg.vocab);
    state_slots = cfg.has_state() ? r->opt.max_num_seqs : 0;
    const size_t T = (size_t)std::max(r->opt.max_num_batched_tokens, r->opt.max_num_seqs);
    const size_t slots = (size_t)r->opt.num_kvcache_blocks * r->opt.kvcache_block_size;
    int rc;
    L.resize(cfg.layers.size());
    size_t m_np = 0, m_ow = 0, m_ff = 0, m_dqk = 0, m_dv = 0, m_gb = 0;
    int64_t wbytes = 0;
    const int W = cfg.width;
    for (size_t i = 0; i < cfg.layers.size(); ++i) {
      const auto& ly = cfg.layers[i];
      FLayerW& w = L[i];
      const std::string p = "l" + std::to_string(i) + ".";
      if ((rc = zalloc(r, &w.n1, W * 4)) || (rc = zalloc(r, &w.n1b, W * 4))) return rc;
      want[p + "norm1"] = false;
      want[p + "norm1b"] = false;
      int ow = 0;
      if (ly.kind == nvc_fefozen_layer::Latent) {
        const auto& a = ly.lat;
        int cols = 0;
        int64_t wn = 0;
        if ((rc = latent_init(r, a, p, slots, 0, w.lat, &cols, &wn))) return rc;
        w.g_off = cols;
        ow = a.heads * a.vdim;
        w.np = pad64(w.g_off + ow);
        for (const char* n : {"mix.g", "mix.o"}) want[p + n] = false;
        wbytes += (int64_t)esz * ((int64_t)(cols + ow) * W + wn + (int64_t)W * ow);
      } else {
        const auto& d = ly.delta;
        const int qk = d.kv_heads * d.dim, vw = d.heads * d.vdim, C = 2 * qk + vw;
        w.q_off = 0; w.k_off = qk; w.v_off = 2 * qk; w.b_off = C; w.a_off = C + d.heads; w.g_off = C + 2 * d.heads;
        ow = vw;
        w.np = pad64(w.g_off + vw);
        if ((rc = zalloc(r, &w.conv_w, (size_t)C * d.taps * 4)) || (rc = zalloc(r, &w.conv_state, (size_t)state_slots * std::max(d.taps - 1, 1) * C * 4)) ||
            (rc = zalloc(r, &w.A_log, d.heads * 4)) || (rc = zalloc(r, &w.dt_bias, d.heads * 4)) || (rc = zalloc(r, &w.onorm, d.vdim * 4)) ||
            (rc = zalloc(r, &w.state, (size_t)state_slots * d.heads * d.dim * d.vdim * 4)))
          return rc;
        for (const char* n : {"mix.q", "mix.q.conv", "mix.k", "mix.k.conv", "mix.v", "mix.v.conv", "mix.b", "mix.a", "mix.A_log", "mix.dt_bias",
                              "mix.norm", "mix.g", "mix.o"})
          want[p + n] = false;
        wbytes += (int64_t)esz * ((int64_t)(C + 2 * d.heads + vw) * W + (int64_t)W * vw);
        m_dqk = std::max(m_dqk, (size_t)qk);
        m_dv = std::max(m_dv, (size_t)vw);
        m_gb = std::max(m_gb, (size_t)2 * d.heads);
      }
      w.owp = pad64(ow);
      if ((rc = zalloc(r, &w.w_in, (size_t)w.np * Wp * esz)) || (rc = zalloc(r, &w.w_o, (size_t)Wp * w.owp * esz))) return rc;
      m_np = std::max(m_np, (size_t)w.np);
      m_ow = std::max(m_ow, (size_t)w.owp);
      const auto& f = ly.mlp;
      if (f.kind != nvc_routed_mlp_spec::None) {
        if ((rc = zalloc(r, &w.n2, W * 4)) || (rc = zalloc(r, &w.n2b, W * 4))) return rc;
        want[p + "norm2"] = false;
        want[p + "norm2b"] = false;
      }
      if (f.kind == nvc_routed_mlp_spec::Dense) {
        w.ffp = pad64(f.ff);
        if ((rc = zalloc(r, &w.w_up, (size_t)w.ffp * Wp * esz)) || (rc = zalloc(r, &w.w_down, (size_t)Wp * w.ffp * esz))) return rc;
        want[p + "mlp.up"] = false;
        want[p + "mlp.down"] = false;
        wbytes += (int64_t)esz * 2 * f.ff * W;
        m_ff = std::max(m_ff, (size_t)w.ffp);
      } else if (f.kind == nvc_routed_mlp_spec::Moe) {
        if ((rc = experts.init(*this, r, f, p, W, T, w.moe, &wbytes))) return rc;
      }
    }
    if ((rc = zalloc(r, &embed, (size_t)Vp * Wp * esz)) || (rc = zalloc(r, &fw, W * 4))) return rc;
    want["embed"] = false;
    want["final.norm"] = false;
    r->weight_bytes = wbytes + (int64_t)esz * cfg.vocab * W;
    // activations (zeroed once: padding columns are never written)
    if ((rc = zalloc(r, &x0, T * Wp * 4)) || (rc = zalloc(r, &res, T * Wp * 4)) || (rc = zalloc(r, &mix, T * Wp * 4)) ||
        (rc = zalloc(r, &ffo, T * Wp * 4)) || (rc = zalloc(r, &proj, T * m_np * 4)) || (rc = zalloc(r, &h, T * Wp * esz)) ||
        (rc = zalloc(r, &ao, T * m_ow * esz)) || (rc = zalloc(r, &hn, (size_t)r->max_logit_rows * Wp * esz)))
      return rc;
    if ((rc = latent_alloc(r, T))) return rc;
    if (m_dv && ((rc = zalloc(r, &rq, T * m_dqk * 4)) || (rc = zalloc(r, &rk, T * m_dqk * 4)) || (rc = zalloc(r, &rv, T * m_dv * 4)) ||
                 (rc = zalloc(r, &ro, T * m_dv * 4)) || (rc = zalloc(r, &gb, T * m_gb * 4))))
      return rc;
    if (m_ff && (rc = zalloc(r, &act, T * m_ff * esz))) return rc;
    if ((rc = experts.alloc(*this, r, Wp, T))) return rc;
    return NVC_OK;
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
    const int W = cfg.width;
    auto vec = [&](float* dst, size_t len) { return n == len ? put_f32(r, dst, v.data(), len) : bad(); };
    int rc = NVC_OK;
    if (name == "embed") { if (!shape_is(cfg.vocab, W)) return bad(); rc = put_matrix(r, embed, Wp, 0, 0, v.data(), cfg.vocab, W, W, 1); }
    else if (name == "final.norm") rc = vec(fw, W);
    else {
      const size_t dot = name.find('.');
      const int li = atoi(name.substr(1, dot - 1).c_str());
      const std::string sub = name.substr(dot + 1);
      const auto& ly = cfg.layers[li];
      const auto& a = ly.lat;
      const auto& d = ly.delta;
      const auto& f = ly.mlp;
      FLayerW& w = L[li];
      const bool latent = ly.kind == nvc_fefozen_layer::Latent;
      auto in_rows = [&](int off, int rows) { return shape_is(rows, W) ? put_matrix(r, w.w_in, Wp, off, 0, v.data(), rows, W, W, 1) : bad(); };
      const int ow = latent ? a.heads * a.vdim : d.heads * d.vdim;
      const int qk = d.kv_heads * d.dim;
      if (latent) {
        bool taken = false;
        rc = latent_load(r, a, w.lat, sub, v, d0, d1, in_rows, bad, &taken);
        if (taken) {
          it->second = rc == NVC_OK;
          return rc;
        }
      }
      {
        bool taken = false;
        rc = experts.load(*this, r, f, W, w.moe, sub, v, d0, d1, bad, &taken);
        if (taken) {
          it->second = rc == NVC_OK;
          return rc;
        }
      }
      if (sub == "norm1") rc = vec(w.n1, W);
      else if (sub == "norm1b") rc = vec(w.n1b, W);
      else if (sub == "norm2") rc = vec(w.n2, W);
      else if (sub == "norm2b") rc = vec(w.n2b, W);
      else if (sub == "mix.g") rc = in_rows(w.g_off, ow);
      else if (sub == "mix.o") { if (!shape_is(W, ow)) return bad(); rc = put_matrix(r, w.w_o, w.owp, 0, 0, v.data(), W, ow, ow, 1); }
      else if (!latent && sub == "mix.q") rc = in_rows(w.q_off, qk);
      else if (!latent && sub == "mix.k") rc = in_rows(w.k_off, qk);
      else if (!latent && sub == "mix.v") rc = in_rows(w.v_off, ow);
      else if (!latent && sub == "mix.b") rc = in_rows(w.b_off, d.heads);
      else if (!latent && sub == "mix.a") rc = in_rows(w.a_off, d.heads);
      else if (!latent && (sub == "mix.q.conv" || sub == "mix.k.conv" || sub == "mix.v.conv")) {
        // [channels, taps] of the checkpoint -> tap-major [taps, all channels] (q, k, v side by side): a warp's lanes read neighbours
        const int rows = sub == "mix.v.conv" ? ow : qk, ch0 = sub == "mix.q.conv" ? 0 : (sub == "mix.k.conv" ? qk : 2 * qk), C = 2 * qk + ow;
        if (!shape_is(rows, d.taps)) return bad();
        std::vector<float> col(rows);
        for (int i = 0; i < d.taps && rc == NVC_OK; ++i) {
          for (int c = 0; c < rows; ++c) col[c] = v[(size_t)c * d.taps + i];
          rc = put_f32(r, w.conv_w + (size_t)i * C + ch0, col.data(), rows);
        }
      }
      else if (!latent && sub == "mix.A_log") rc = vec(w.A_log, d.heads);
      else if (!latent && sub == "mix.dt_bias") rc = vec(w.dt_bias, d.heads);
      else if (!latent && sub == "mix.norm") rc = vec(w.onorm, d.vdim);
      else if (sub == "mlp.up") { if (!shape_is(f.ff, W)) return bad(); rc = put_matrix(r, w.w_up, Wp, 0, 0, v.data(), f.ff, W, W, 1); }
      else if (sub == "mlp.down") { if (!shape_is(W, f.ff)) return bad(); rc = put_matrix(r, w.w_down, w.ffp, 0, 0, v.data(), W, f.ff, f.ff, 1); }
    }
    if (rc == NVC_OK) it->second = true;
    return rc;
  }

  int finalize(nvc_runner* r) override {
    return require_all_tensors(r);
  }

  int tap(nvc_runner* r, int run, int N) { return copy_tap(r, res, Wp, tap_host, tap_cap, run, N, cfg.width); }

  int latent_mixer(nvc_runner* r, const nvc_step_shape& s, int li) {
    const auto& a = cfg.layers[li].lat;
    FLayerW& w = L[li];
    return latent_run(r, s, a, w.lat, a.kv_from < 0 ? w.lat : L[a.kv_from].lat, cfg.eps, proj, w.np, proj + w.g_off, ao, w.owp);
  }

  int delta_mixer(nvc_runner* r, const nvc_step_shape& s, int li) {
    nvc_ctx* ctx = r->ctx;
    void* st = r->stream;
    const auto& d = cfg.layers[li].delta;
    FLayerW& w = L[li];
    nvc_delta_prep p{};
    p.in = proj; p.ldi = w.np;
    p.q_off = w.q_off; p.k_off = w.k_off; p.v_off = w.v_off; p.b_off = w.b_off; p.a_off = w.a_off;
    p.heads = d.heads; p.kv_heads = d.kv_heads; p.dim = d.dim; p.vdim = d.vdim; p.taps = d.taps;
    p.conv_w = w.conv_w; p.conv_state = w.conv_state;
    p.state_slots = r->d_state_slots; p.cu_seqlens = s.decode ? nullptr : r->d_cu; p.positions = r->d_pos;
    p.A_log = w.A_log; p.dt_bias = w.dt_bias;
    p.unit_eps = kUnitEps; p.q_scale = 1.0f / sqrtf((float)d.dim);
    p.q_out = rq; p.k_out = rk; p.v_out = rv; p.ldq = p.ldk = d.kv_heads * d.dim; p.ldv = d.heads * d.vdim;
    p.gb_out = gb;
    p.B = s.B;
    int rc = nvc_delta_prep_run(ctx, &p, s.N, s.decode ? 1 : s.max_seqlen, st);
    if (rc) return rc;
    mark(r, "delta_prep");
    if ((rc = nvc_delta_rule_scan(ctx, &p, ro, p.ldv, w.state, s.decode ? 1 : s.max_seqlen, st))) return rc;
    mark(r, "delta_scan");
    rc = nvc_head_gate_w(ctx, ro, p.ldv, proj + w.g_off, w.np, w.onorm, ao, w.owp, dt, d.heads, d.vdim, 1, cfg.eps, NVC_GATE_SILU, 1.f, s.N, st);
    mark(r, "head_gate");
    return rc;
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
    const float* pend = nullptr;       // a sublayer's output whose norm and residual sum are still to come
    const float* pend_w = nullptr;
    for (size_t i = 0; i < cfg.layers.size(); ++i) {
      const auto& ly = cfg.layers[i];
      FLayerW& w = L[i];
      const bool first = i == 0;
      if (tap_host && !first) {
        // debug: land the previous layer's last sum first, copy the stream out, then open this layer
        if ((rc = nvc_rms_norm_sandwich(ctx, res, pend, pend_w, res, Wp, nullptr, nullptr, dt, 0, cfg.eps, 1.f, nullptr, N, W, st))) return rc;
        if ((rc = tap(r, (int)i - 1, N))) return rc;
        pend = pend_w = nullptr;
      }
      if ((rc = nvc_rms_norm_sandwich(ctx, first ? x0 : res, pend, pend_w, res, Wp, w.n1, h, dt, Wp, cfg.eps, 1.f, nullptr, N, W, st))) return rc;
      mark(r, "norm");
      // ---- mixer
      if ((rc = linear(r, h, Wp, w.w_in, proj, w.np, NVC_DT_F32, N, w.np, Wp))) return rc;
      mark(r, "gemm_in");
      if ((rc = ly.kind == nvc_fefozen_layer::Latent ? latent_mixer(r, s, (int)i) : delta_mixer(r, s, (int)i))) return rc;
      if ((rc = linear(r, ao, w.owp, w.w_o, mix, Wp, NVC_DT_F32, N, Wp, w.owp))) return rc;
      mark(r, "gemm_o");
      pend = mix;
      pend_w = w.n1b;
      // ---- feed-forward
      const auto& f = ly.mlp;
      if (f.kind == nvc_routed_mlp_spec::None) continue;
      if ((rc = nvc_rms_norm_sandwich(ctx, res, pend, pend_w, res, Wp, w.n2, h, dt, Wp, cfg.eps, 1.f, nullptr, N, W, st))) return rc;
      mark(r, "norm");
      if (f.kind == nvc_routed_mlp_spec::Dense) {
        if (use_tc) {        // tanh-gelu in the epilogue of the up-projection
          if ((rc = nvc_gemm_bf16_act(ctx, reinterpret_cast<const nvc_bf16*>(h), Wp, reinterpret_cast<const nvc_bf16*>(w.w_up), act, w.ffp, NVC_DT_BF16,
                                      N, w.ffp, Wp, NVC_ACT_GELU_TANH, st)))
            return rc;
        } else if ((rc = linear(r, h, Wp, w.w_up, act, w.ffp, dt, N, w.ffp, Wp, NVC_ACT_GELU_TANH))) {
          return rc;
        }
        mark(r, "gemm_up");
        if ((rc = linear(r, act, w.ffp, w.w_down, ffo, Wp, NVC_DT_F32, N, Wp, w.ffp))) return rc;
        mark(r, "gemm_down");
      } else if ((rc = experts.run(*this, r, f, w.moe, h, ffo, N, W))) {
        return rc;
      }
      pend = ffo;
      pend_w = w.n2b;
    }
    if (tap_host) {
      if ((rc = nvc_rms_norm_sandwich(ctx, res, pend, pend_w, res, Wp, nullptr, nullptr, dt, 0, cfg.eps, 1.f, nullptr, N, W, st))) return rc;
      if ((rc = tap(r, (int)cfg.layers.size() - 1, N))) return rc;
      pend = pend_w = nullptr;
      tap_host = nullptr;      // one step only
    }
    // ---- head: the last sum and the final norm of the wanted rows, logits against the embedding table
    rc = nvc_rms_norm_sandwich(ctx, res, pend, pend_w, nullptr, Wp, fw, hn, dt, Wp, cfg.eps, 1.f, s.decode ? nullptr : r->d_last_rows, s.rows, W, st);
    if (rc) return rc;
    mark(r, "final_norm");
    rc = linear(r, hn, Wp, embed, r->logits, Vp, NVC_DT_F32, s.rows, Vp, Wp);
    mark(r, "lm_head");
    finish_profile(r);
    return rc;
  }
};

}  // namespace

nvc_model_body* nvc_make_fefozen_body(nvc_runner* r, const nvc_fefozen_config& cfg, int* status) {
  FefozenBody* b = new FefozenBody();
  b->cfg = cfg;
  *status = b->init(r);
  return b;
}
