// A routed mixture of experts as a feed-forward, for the model bodies that have it (Fefozen, Vizotar): sizes, weights, loading and the
// launches of a step.
//   router product (fp32 out) -> nvc_moe_route_logits_ex -> counting sort by expert -> grouped [gate; up] product -> gated unit ->
//   grouped down product (fp32) -> nvc_moe_combine (or with identity experts, which add the token's own row)
// With bf16 storage and expert widths of 128 and more the grouped products run on the tcgen05 kernel over groups padded to 128 rows,
// else on the generic grouped kernel.
#pragma once
#include <algorithm>
#include <string>
#include <vector>

#include "body_common.h"

namespace {

struct nvc_experts_weights {
  void* router = nullptr;               // [Ep, Wp]
  float* bias = nullptr;                // [experts]: what the router adds to scores or logits
  int Ep = 0, effp = 0;
  void *w_egu = nullptr, *w_edown = nullptr;   // [E][2 effp, Wp] (gate rows, then up rows at effp), [E][Wp, effp]
  bool tc = false;
};

// how a family routes and what its experts compute
struct nvc_experts_kind {
  const char* bias_name;                // tensor of the router's bias / correction
  int score, normalize;                 // nvc_moe_route_logits_ex
  int act;                              // NVC_ACT_GLU_CLAMP or NVC_ACT_SILU_MUL
  float alpha;                          // NVC_ACT_GLU_CLAMP (its limit comes from the layer)
};

struct nvc_experts {
  nvc_experts_kind kind;
  bool use_tc = true;                   // tcgen05 for the grouped products
  // activations
  float *zlog = nullptr, *tk_w = nullptr, *y = nullptr;
  void *hid2 = nullptr, *hid = nullptr, *xs = nullptr;
  int32_t *tk_idx = nullptr, *offsets = nullptr, *src_rows = nullptr, *pos = nullptr, *tile_group = nullptr;
  size_t m_Ep = 0, m_top = 0, m_E = 0, m_hid = 0, m_rows = 0, m_tiles = 0;

  static int tiles(int pairs, int experts) { return (pairs + experts * 127 + 127) / 128; }

  // weights of one layer (tensors p + "mlp...."); T: rows of the longest step
  int init(nvc_body_base& b, nvc_runner* r, const nvc_routed_mlp_spec& f, const std::string& p, int W, size_t T, nvc_experts_weights& w, int64_t* weights) {
    const int Et = f.experts + f.identity, Wp = pad64(W);
    w.Ep = pad64(Et);
    w.effp = pad64(f.expert_ff);
    w.tc = use_tc && f.experts > 0 && w.effp >= 128;
    int rc;
    if ((rc = b.zalloc(r, &w.router, (size_t)w.Ep * Wp * b.esz)) || (rc = b.zalloc(r, &w.bias, Et * 4))) return rc;
    b.want[p + "mlp.router"] = false;
    b.want[p + kind.bias_name] = false;
    if (f.experts > 0 && ((rc = b.zalloc(r, &w.w_egu, (size_t)f.experts * 2 * w.effp * Wp * b.esz)) ||
                          (rc = b.zalloc(r, &w.w_edown, (size_t)f.experts * Wp * w.effp * b.esz))))
      return rc;
    for (int e = 0; e < f.experts; ++e)
      for (const char* n : {"gate", "up", "down"}) b.want[p + "mlp.e" + std::to_string(e) + "." + n] = false;
    *weights += (int64_t)b.esz * ((int64_t)Et * W + (int64_t)f.experts * 3 * f.expert_ff * W);
    m_Ep = std::max(m_Ep, (size_t)w.Ep);
    m_top = std::max(m_top, (size_t)f.top);
    m_E = std::max(m_E, (size_t)Et);
    m_hid = std::max(m_hid, (size_t)w.effp);
    m_rows = std::max(m_rows, w.tc ? (size_t)tiles((int)T * f.top, Et) * 128 : T * f.top);
    if (w.tc) m_tiles = std::max(m_tiles, (size_t)tiles((int)T * f.top, Et));
    return NVC_OK;
  }

  // activations of the widest layer (zeroed once: padding columns are never written)
  int alloc(nvc_body_base& b, nvc_runner* r, int Wp, size_t T) {
    if (!m_E) return NVC_OK;
    int rc;
    if ((rc = b.zalloc(r, &zlog, T * m_Ep * 4)) || (rc = b.zalloc(r, &tk_idx, T * m_top * 4)) || (rc = b.zalloc(r, &tk_w, T * m_top * 4)) ||
        (rc = b.zalloc(r, &offsets, (m_E + 1) * 4)) || (rc = b.zalloc(r, &src_rows, m_rows * 4)) || (rc = b.zalloc(r, &pos, T * m_top * 4)) ||
        (rc = b.zalloc(r, &hid2, m_rows * 2 * m_hid * b.esz)) || (rc = b.zalloc(r, &hid, m_rows * m_hid * b.esz)) ||
        (rc = b.zalloc(r, &y, m_rows * Wp * 4)))
      return rc;
    if (m_tiles && ((rc = b.zalloc(r, &tile_group, m_tiles * 4)) || (rc = b.zalloc(r, &xs, m_rows * Wp * b.esz)))) return rc;
    return NVC_OK;
  }

  // one tensor `sub` ("mlp....") of a layer; *taken = false when it is not one of the experts'
  template <typename Bad>
  int load(nvc_body_base& b, nvc_runner* r, const nvc_routed_mlp_spec& f, int W, nvc_experts_weights& w, const std::string& sub, const std::vector<float>& v,
           int64_t d0, int64_t d1, Bad&& bad, bool* taken) {
    const int Et = f.experts + f.identity, Wp = pad64(W);
    *taken = f.kind == nvc_routed_mlp_spec::Moe;
    if (!*taken) return NVC_OK;
    auto is = [&](int64_t rows, int64_t cols) { return d0 == rows && d1 == cols; };
    if (sub == "mlp.router") return is(Et, W) ? b.put_matrix(r, w.router, Wp, 0, 0, v.data(), Et, W, W, 1) : bad();
    if (sub == kind.bias_name) return (int)v.size() == Et ? b.put_f32(r, w.bias, v.data(), Et) : bad();
    const size_t dot = sub.rfind("mlp.e", 0) == 0 ? sub.find('.', 5) : std::string::npos;
    if (dot == std::string::npos) { *taken = false; return NVC_OK; }
    const int e = atoi(sub.substr(5, dot - 5).c_str());
    const std::string part = sub.substr(dot + 1);
    if (part == "down")
      return is(W, f.expert_ff) ? b.put_matrix(r, reinterpret_cast<uint8_t*>(w.w_edown) + (size_t)e * Wp * w.effp * b.esz, w.effp, 0, 0, v.data(), W,
                                               f.expert_ff, f.expert_ff, 1)
                                : bad();
    uint8_t* gu = reinterpret_cast<uint8_t*>(w.w_egu) + (size_t)e * 2 * w.effp * Wp * b.esz;
    return is(f.expert_ff, W) ? b.put_matrix(r, gu, Wp, part == "up" ? w.effp : 0, 0, v.data(), f.expert_ff, W, W, 1) : bad();
  }

  // out[:N, :W] = the weighted sum of the chosen experts' outputs of h (rows in the storage format)
  int run(nvc_body_base& b, nvc_runner* r, const nvc_routed_mlp_spec& f, const nvc_experts_weights& w, const void* h, float* out, int N, int W) {
    nvc_ctx* ctx = r->ctx;
    void* st = r->stream;
    const int Wp = pad64(W), Et = f.experts + f.identity, P = N * f.top, dt = b.dt;
    int rc;
    if (b.use_tc) {
      if ((rc = b.linear(r, h, Wp, w.router, zlog, w.Ep, NVC_DT_F32, N, w.Ep, Wp))) return rc;
    } else if ((rc = nvc_linear(ctx, h, Wp, 0, w.router, Wp, 0, zlog, w.Ep, 0, dt, NVC_DT_F32, N, Et, Wp, 1, NVC_ACT_NONE, st))) {
      return rc;
    }
    if ((rc = nvc_moe_route_logits_ex(ctx, zlog, w.Ep, w.bias, Et, f.top, 1.f, -1, kind.score, kind.normalize, tk_idx, tk_w, nullptr, N, st))) return rc;
    b.mark(r, "moe_route");
    if (w.tc) {
      const int nt = tiles(P, Et), mcap = nt * 128;
      if ((rc = nvc_moe_sort_padded_ex(ctx, tk_idx, N, f.top, Et, f.experts, 128, offsets, src_rows, pos, tile_group, nt, st))) return rc;
      b.mark(r, "moe_sort");
      if ((rc = nvc_gather_rows_bf16(ctx, reinterpret_cast<const nvc_bf16*>(h), Wp, src_rows, offsets + f.experts, reinterpret_cast<nvc_bf16*>(xs), Wp,
                                     mcap, Wp, st)))
        return rc;
      b.mark(r, "moe_gather");
      if ((rc = nvc_gemm_bf16_grouped(ctx, reinterpret_cast<const nvc_bf16*>(xs), Wp, reinterpret_cast<const nvc_bf16*>(w.w_egu), hid2, 2 * w.effp,
                                      NVC_DT_BF16, mcap, 2 * w.effp, Wp, tile_group, f.experts, NVC_ACT_NONE, st)))
        return rc;
      b.mark(r, "moe_gate_up");
      if ((rc = nvc_act_mul_p(ctx, hid2, 2 * w.effp, hid, w.effp, dt, mcap, f.expert_ff, w.effp, kind.act, f.limit, kind.alpha, st))) return rc;
      b.mark(r, "moe_glu");
      if ((rc = nvc_gemm_bf16_grouped(ctx, reinterpret_cast<const nvc_bf16*>(hid), w.effp, reinterpret_cast<const nvc_bf16*>(w.w_edown), y, Wp, NVC_DT_F32,
                                      mcap, Wp, w.effp, tile_group, f.experts, NVC_ACT_NONE, st)))
        return rc;
      b.mark(r, "moe_down");
    } else {
      if ((rc = nvc_moe_sort(ctx, tk_idx, N, f.top, Et, offsets, src_rows, pos, st))) return rc;
      b.mark(r, "moe_sort");
      if (f.experts > 0) {
        if ((rc = nvc_linear_grouped(ctx, h, Wp, src_rows, w.w_egu, Wp, (int64_t)2 * w.effp * Wp, hid2, 2 * w.effp, offsets, f.experts, P, dt, dt,
                                     2 * w.effp, Wp, NVC_ACT_NONE, st)))
          return rc;
        b.mark(r, "moe_gate_up");
        if ((rc = nvc_act_mul_p(ctx, hid2, 2 * w.effp, hid, w.effp, dt, P, f.expert_ff, w.effp, kind.act, f.limit, kind.alpha, st))) return rc;
        b.mark(r, "moe_glu");
        if ((rc = nvc_linear_grouped(ctx, hid, w.effp, nullptr, w.w_edown, w.effp, (int64_t)Wp * w.effp, y, Wp, offsets, f.experts, P, dt, NVC_DT_F32, Wp,
                                     w.effp, NVC_ACT_NONE, st)))
          return rc;
        b.mark(r, "moe_down");
      }
    }
    if (f.identity > 0) rc = nvc_moe_combine_identity(ctx, y, NVC_DT_F32, Wp, pos, tk_w, tk_idx, f.top, f.experts, h, dt, Wp, out, Wp, N, W, st);
    else rc = nvc_moe_combine(ctx, y, NVC_DT_F32, Wp, pos, tk_w, f.top, nullptr, NVC_DT_F32, 0, nullptr, out, Wp, N, W, st);
    b.mark(r, "moe_combine");
    return rc;
  }
};

}  // namespace
