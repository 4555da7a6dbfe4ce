// Buzutar model body behind the step executor (runner.cu): weights, paged pools of shared key / value rows, the layer loop.
//
// One layer over the N query rows of a step (x <- x + n1(mixer(x)); x <- x + n2(ff(x)); the sublayers read x itself):
//   nvc_rms_norm_sandwich     x += norm(previous sublayer's output); h = x in the storage format: one pass over the row
//   sigmoid attention:
//     linear w_in             [q | k | gate], fp32 out
//     nvc_qk_norm_fold_store  norms over the whole query and the whole key projection, query temperature; the key norm's weight meets
//                             the queries and its root mean square travels as one number per token, so that a token leaves ONE row -
//                             its projected key, which is its value too - in this layer's paged pool
//     attention               sigmoid(score + bias) weights over all cached rows, output gate in the epilogue: nvc_attn_paged_wide, or the
//                             tcgen05 paged-prefill kernel for long portions when heads have 128 numbers (each row loaded once)
//   latent attention:
//     linear w_in             [dq | dkv], fp32 out
//     latent_run              (latent_mixer.h) latents, absorbed queries, windowed attention over shared rows, value up-projection
//   linear o
//   feed-forward: linear up with the squared relu in its epilogue -> linear down (fp32)
// The residual sum itself happens in the NEXT nvc_rms_norm_sandwich (or the final one), in fp32.
//
// Feature dimensions that a dense matrix product sums over or produces are padded to multiples of 64 in the weight and activation
// buffers (zeros), so that the tcgen05 GEMMs (K % 64, N % 16) take every such product of the bf16 mode; heads are not padded.
#include <cmath>
#include <cstring>
#include <string>
#include <vector>

#include "latent_mixer.h"
#include "runner.h"

namespace {

struct BLayerW {
  float *n1 = nullptr, *n2 = nullptr;
  void* w_in = nullptr;                 // [np, Wp]
  int np = 0;
  nvc_latent_weights lat;
  // sigmoid attention
  int k_off = 0, g_off = 0, qw = 0, kw = 0, ldq = 0, ldpool = 0;
  std::vector<float> q_norm, k_norm;    // host copies until finalize() folds them
  float *wqk = nullptr, *pb = nullptr, *key_scale = nullptr;
  void* pool = nullptr;                 // [slots, ldpool]: a token's projected keys
  void* w_o = nullptr;                  // [Wp, owp]
  int owp = 0;
  void *w_up = nullptr, *w_down = nullptr;
  int ffp = 0;
};

struct BuzutarBody : nvc_latent_body {
  nvc_buzutar_config cfg;
  int Wp = 0, Vp = 0;
  std::vector<BLayerW> L;
  void *embed = nullptr, *head = nullptr;
  float* fw = nullptr;
  // activations
  float *x0 = nullptr, *res = nullptr, *proj = nullptr, *mix = nullptr, *ffo = nullptr;
  void *h = nullptr, *q = nullptr, *ao = nullptr, *act = nullptr, *hn = nullptr;
  float* tap_host = nullptr;
  size_t tap_cap = 0;

  int vocab() const override { return cfg.vocab; }
  int logits_ld() const override { return Vp; }
  int layer_runs() const override { return (int)cfg.layers.size(); }
  int width() const override { return cfg.width; }
  int64_t cache_bytes_per_token() const override {
    int64_t b = 0;
    for (size_t i = 0; i < cfg.layers.size(); ++i) {
      if (cfg.layers[i].kind == nvc_buzutar_layer::Attention) b += (int64_t)L[i].ldpool * (int64_t)esz + 4;
      else if (cfg.layers[i].lat.kv_from < 0) b += (int64_t)L[i].lat.ldpool * (int64_t)esz;
    }
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
    use_tc = dt == NVC_DT_BF16 && !(getenv("NVC_BUZUTAR_TC") && atoi(getenv("NVC_BUZUTAR_TC")) == 0);
    use_flash = use_tc && !(getenv("NVC_BUZUTAR_FLASH") && atoi(getenv("NVC_BUZUTAR_FLASH")) == 0);
    Wp = pad64(cfg.width);
    Vp = pad64(cfg.vocab);
    const size_t T = (size_t)std::max(r->opt.max_num_batched_tokens, r->opt.max_num_seqs);
    const size_t slots = (size_t)r->opt.num_kvcache_blocks * r->opt.kvcache_block_size;
    const int W = cfg.width;
    NVC_REQUIRE(ctx, W <= 12288, NVC_ESHAPE, "width above 12 288");
    int rc;
    L.resize(cfg.layers.size());
    size_t m_np = 0, m_q = 0, m_ow = 0, m_ff = 0;
    int64_t wbytes = 0;
    for (size_t i = 0; i < cfg.layers.size(); ++i) {
      const auto& ly = cfg.layers[i];
      BLayerW& w = L[i];
      const std::string p = "l" + std::to_string(i) + ".";
      if ((rc = zalloc(r, &w.n1, W * 4))) return rc;
      want[p + "norm1"] = false;
      int ow = 0, cols = 0;
      if (ly.kind == nvc_buzutar_layer::Latent) {
        int64_t wn = 0;
        if ((rc = latent_init(r, ly.lat, p, slots, 0, w.lat, &cols, &wn))) return rc;
        ow = ly.lat.heads * ly.lat.vdim;
        wbytes += (int64_t)esz * wn;
      } else {
        const auto& a = ly.attn;
        NVC_REQUIRE(ctx, a.dim <= 512, NVC_ESHAPE, "attention heads above 512 numbers");
        ow = w.qw = a.heads * a.dim;
        w.kw = a.kv_heads * a.dim;
        w.k_off = w.qw;
        w.g_off = w.qw + w.kw;
        cols = w.g_off + ow;
        w.ldq = pad8(w.qw);
        w.ldpool = pad8(w.kw);
        if ((rc = zalloc(r, &w.wqk, w.qw * 4)) || (rc = zalloc(r, &w.pb, a.heads * 4)) || (rc = zalloc(r, &w.key_scale, slots * 4)) ||
            (rc = zalloc(r, &w.pool, slots * w.ldpool * esz)))
          return rc;
        for (const char* n : {"mix.q", "mix.k", "mix.q.norm", "mix.k.norm", "mix.pb", "mix.g"}) want[p + n] = false;
        m_q = std::max(m_q, (size_t)w.ldq);
      }
      want[p + "mix.o"] = false;
      w.np = pad64(cols);
      w.owp = pad64(ow);
      if ((rc = zalloc(r, &w.w_in, (size_t)w.np * Wp * esz)) || (rc = zalloc(r, &w.w_o, (size_t)Wp * w.owp * esz))) return rc;
      wbytes += (int64_t)esz * (cols + ow) * W;
      m_np = std::max(m_np, (size_t)w.np);
      m_ow = std::max(m_ow, (size_t)w.owp);
      if (ly.ff > 0) {
        w.ffp = pad64(ly.ff);
        if ((rc = zalloc(r, &w.n2, W * 4)) || (rc = zalloc(r, &w.w_up, (size_t)w.ffp * Wp * esz)) || (rc = zalloc(r, &w.w_down, (size_t)Wp * w.ffp * esz)))
          return rc;
        for (const char* n : {"norm2", "mlp.up", "mlp.down"}) want[p + n] = false;
        wbytes += (int64_t)esz * 2 * ly.ff * W;
        m_ff = std::max(m_ff, (size_t)w.ffp);
      }
    }
    if ((rc = zalloc(r, &embed, (size_t)Vp * Wp * esz)) || (rc = zalloc(r, &head, (size_t)Vp * Wp * esz)) || (rc = zalloc(r, &fw, W * 4))) return rc;
    want["embed"] = want["head"] = want["final.norm"] = false;
    r->weight_bytes = wbytes + (int64_t)esz * cfg.vocab * W;      // the head; of the embedding a step reads single rows
    // activations (zeroed once: padding columns are never written)
    if ((rc = zalloc(r, &x0, T * Wp * 4)) || (rc = zalloc(r, &res, T * Wp * 4)) || (rc = zalloc(r, &mix, T * Wp * 4)) || (rc = zalloc(r, &ffo, T * Wp * 4)) ||
        (rc = zalloc(r, &proj, T * m_np * 4)) || (rc = zalloc(r, &h, T * Wp * esz)) || (rc = zalloc(r, &ao, T * m_ow * esz)) ||
        (rc = zalloc(r, &hn, (size_t)r->max_logit_rows * Wp * esz)))
      return rc;
    if (m_q && (rc = zalloc(r, &q, T * m_q * esz))) return rc;
    if (m_ff && (rc = zalloc(r, &act, T * m_ff * esz))) return rc;
    return latent_alloc(r, T);
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
    auto shape_is = [&](int64_t a, int64_t b) { return ndim == 2 && d0 == a && d1 == b; };
    auto bad = [&]() {
      nvc_set_error(ctx, "unexpected shape for " + name);
      return NVC_ESHAPE;
    };
    const int W = cfg.width;
    auto vec = [&](float* dst, size_t len) { return n == len ? put_f32(r, dst, v.data(), len) : bad(); };
    auto keep = [&](std::vector<float>& dst, size_t len) {
      if (n == len) dst = v;
      return n == len ? NVC_OK : bad();
    };
    auto matrix = [&](void* dst, int ld, int rows, int cols) { return shape_is(rows, cols) ? put_matrix(r, dst, ld, 0, 0, v.data(), rows, cols, cols, 1) : bad(); };
    int rc = NVC_OK;
    if (name == "embed") rc = matrix(embed, Wp, cfg.vocab, W);
    else if (name == "head") rc = matrix(head, Wp, cfg.vocab, W);
    else if (name == "final.norm") rc = vec(fw, W);
    else {
      const size_t dot = name.find('.');
      const int li = atoi(name.substr(1, dot - 1).c_str());
      const std::string sub = name.substr(dot + 1);
      const auto& ly = cfg.layers[li];
      BLayerW& w = L[li];
      const bool latent = ly.kind == nvc_buzutar_layer::Latent;
      auto in_rows = [&](int off, int rows) { return shape_is(rows, W) ? put_matrix(r, w.w_in, Wp, off, 0, v.data(), rows, W, W, 1) : bad(); };
      const int ow = latent ? ly.lat.heads * ly.lat.vdim : w.qw;
      bool taken = false;
      if (latent) rc = latent_load(r, ly.lat, w.lat, sub, v, d0, d1, in_rows, bad, &taken);
      if (!taken) {
        if (sub == "norm1") rc = vec(w.n1, W);
        else if (sub == "norm2") rc = vec(w.n2, W);
        else if (sub == "mix.o") rc = matrix(w.w_o, w.owp, W, ow);
        else if (sub == "mix.q") rc = in_rows(0, w.qw);
        else if (sub == "mix.k") rc = in_rows(w.k_off, w.kw);
        else if (sub == "mix.g") rc = in_rows(w.g_off, ow);
        else if (sub == "mix.q.norm") rc = keep(w.q_norm, w.qw);
        else if (sub == "mix.k.norm") rc = keep(w.k_norm, w.kw);
        else if (sub == "mix.pb") rc = vec(w.pb, ly.attn.heads);
        else if (sub == "mlp.up") rc = matrix(w.w_up, Wp, ly.ff, W);
        else if (sub == "mlp.down") rc = matrix(w.w_down, w.ffp, W, ly.ff);
      }
    }
    if (rc == NVC_OK) it->second = true;
    return rc;
  }

  int finalize(nvc_runner* r) override {
    int rc = require_all_tensors(r);
    if (rc) return rc;
    for (size_t i = 0; i < cfg.layers.size(); ++i) {
      if (cfg.layers[i].kind != nvc_buzutar_layer::Attention) continue;
      const auto& a = cfg.layers[i].attn;
      BLayerW& w = L[i];
      const int group = a.heads / a.kv_heads;
      std::vector<float> f(w.qw);
      for (int c = 0; c < w.qw; ++c) f[c] = w.q_norm[c] * w.k_norm[(c / a.dim / group) * a.dim + c % a.dim];
      if ((rc = put_f32(r, w.wqk, f.data(), f.size()))) return rc;
    }
    return NVC_OK;
  }

  int attention_mixer(nvc_runner* r, const nvc_step_shape& s, int li) {
    const auto& a = cfg.layers[li].attn;
    BLayerW& w = L[li];
    int rc = nvc_qk_norm_fold_store(r->ctx, proj, w.np, 0, w.qw, w.k_off, w.kw, w.wqk, cfg.eps, r->d_pos, a.temp_coef, a.temp_every, q, w.ldq, w.pool,
                                    w.ldpool, w.key_scale, r->d_slots, dt, s.N, r->stream);
    if (rc) return rc;
    mark(r, "qk_norm_store");
    nvc_attn_spec sp{};
    sp.heads = a.heads; sp.kv_heads = a.kv_heads; sp.dim = a.dim; sp.vdim = a.dim;
    sp.scale = a.scale;
    sp.gate = proj + w.g_off; sp.ldg = w.np;
    sp.out_scale = 1.f;
    sp.weights = NVC_ATTN_SIGMOID;
    sp.bias = w.pb;
    sp.key_scale = w.key_scale;
    rc = shared_attention(r, s, sp, a.dim == 128 && flash_step(r, s), q, w.ldq, w.pool, w.ldpool, ao, w.owp);
    mark(r, "sigmoid_attention");
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
    int rc = nvc_embed_gather_scaled_f32(ctx, r->d_ids, embed, dt, Wp, cfg.embedding_scale, x0, Wp, N, W, st);
    if (rc) return rc;
    mark(r, "embed");
    const float* pend = nullptr;       // a sublayer's output whose norm and residual sum are still to come
    const float* pend_w = nullptr;
    // lands the pending sum; h = the stream in the storage format (what the next sublayer reads)
    auto land = [&](const float* from, bool with_h) {
      int e = nvc_rms_norm_sandwich(ctx, from, pend, pend_w, res, Wp, nullptr, with_h ? h : nullptr, dt, Wp, cfg.eps, 0.f, nullptr, N, W, st);
      pend = pend_w = nullptr;
      mark(r, "norm");
      return e;
    };
    for (size_t i = 0; i < cfg.layers.size(); ++i) {
      const auto& ly = cfg.layers[i];
      BLayerW& w = L[i];
      if ((rc = land(i == 0 ? x0 : res, true))) return rc;
      if (tap_host && i > 0 && (rc = copy_tap(r, res, Wp, tap_host, tap_cap, (int)i - 1, N, W))) return rc;
      // ---- mixer
      if ((rc = linear(r, h, Wp, w.w_in, proj, w.np, NVC_DT_F32, N, w.np, Wp))) return rc;
      mark(r, "gemm_in");
      if (ly.kind == nvc_buzutar_layer::Latent) {
        const auto& a = ly.lat;
        rc = latent_run(r, s, a, w.lat, a.kv_from < 0 ? w.lat : L[a.kv_from].lat, cfg.eps, proj, w.np, nullptr, ao, w.owp);
      } else {
        rc = attention_mixer(r, s, (int)i);
      }
      if (rc) return rc;
      if ((rc = linear(r, ao, w.owp, w.w_o, mix, Wp, NVC_DT_F32, N, Wp, w.owp))) return rc;
      mark(r, "gemm_o");
      pend = mix;
      pend_w = w.n1;
      // ---- feed-forward
      if (ly.ff == 0) continue;
      if ((rc = land(res, true))) return rc;
      if (use_tc) {        // squared relu in the epilogue of the up-projection
        if ((rc = nvc_gemm_bf16_act(ctx, reinterpret_cast<const nvc_bf16*>(h), Wp, reinterpret_cast<const nvc_bf16*>(w.w_up), act, w.ffp, NVC_DT_BF16, N,
                                    w.ffp, Wp, NVC_ACT_RELU2, st)))
          return rc;
      } else if ((rc = linear(r, h, Wp, w.w_up, act, w.ffp, dt, N, w.ffp, Wp, NVC_ACT_RELU2))) {
        return rc;
      }
      mark(r, "gemm_up");
      if ((rc = linear(r, act, w.ffp, w.w_down, ffo, Wp, NVC_DT_F32, N, Wp, w.ffp))) return rc;
      mark(r, "gemm_down");
      pend = ffo;
      pend_w = w.n2;
    }
    if (tap_host) {
      if ((rc = land(res, false))) return rc;
      if ((rc = copy_tap(r, res, Wp, tap_host, tap_cap, (int)cfg.layers.size() - 1, N, W))) return rc;
      tap_host = nullptr;      // one step only
    }
    // ---- head: the last sum and the final norm of the wanted rows, logits, cap
    rc = nvc_rms_norm_sandwich(ctx, res, pend, pend_w, nullptr, Wp, fw, hn, dt, Wp, cfg.eps, 0.f, s.decode ? nullptr : r->d_last_rows, s.rows, W, st);
    if (rc) return rc;
    mark(r, "final_norm");
    if ((rc = linear(r, hn, Wp, head, r->logits, Vp, NVC_DT_F32, s.rows, Vp, Wp))) return rc;
    mark(r, "lm_head");
    if (cfg.logit_softcap > 0.f) {
      rc = nvc_softcap_f32(ctx, r->logits, Vp, cfg.logit_softcap, s.rows, cfg.vocab, st);
      mark(r, "softcap");
    }
    finish_profile(r);
    return rc;
  }
};

}  // namespace

nvc_model_body* nvc_make_buzutar_body(nvc_runner* r, const nvc_buzutar_config& cfg, int* status) {
  BuzutarBody* b = new BuzutarBody();
  b->cfg = cfg;
  *status = b->init(r);
  return b;
}
