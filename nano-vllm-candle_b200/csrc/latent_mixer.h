// Latent attention with a rotated key part that all heads share, for the model bodies that have it (Fefozen, Buzutar).
//
// Over the N query rows of a step, behind the layer's fused input projection (fp32 rows with [dq | dkv] among their columns):
//   nvc_latent_norm_store_rot  RMS norms of both latents; the token's cache row [normed latent | rotated shared key part] goes
//                              into the layer's paged pool (a layer with kv_from reads the named layer's pool and stores nothing)
//   linear uq (fp32 out) -> nvc_head_split_rot: unrotated query parts, rotated parts straight into the absorbed queries
//   linear uk^T per head       unrotated query parts carried into the latent space (absorbed key up-projection)
//   attention                  softmax over the cached rows: in the absorbed form a layer is multi-query attention with ONE key /
//                              value head - key = the whole row (kv_rank + rot_dim numbers), value = its first kv_rank numbers.
//                              nvc_attn_paged_wide (sink, window), or the tcgen05 paged-prefill kernel for long portions when the
//                              row has 128 numbers (the rotated part rides along as value columns that the value up-projection
//                              never reads)
//   linear uv per head         with a gate: fp32 out -> nvc_head_gate (sigmoid gate of h); without: straight into the mixer's output
#pragma once
#include <map>
#include <string>
#include <tuple>
#include <vector>

#include "body_common.h"
#include "model_config.h"

namespace {

inline int pad8(int v) { return (v + 7) / 8 * 8; }

// what one latent layer keeps on the device
struct nvc_latent_weights {
  int dq_off = 0, kv_off = 0;           // first column of the two down-projections in a projection row
  float *dq_norm = nullptr, *dkv_norm = nullptr, *sink = nullptr;
  void* w_uq = nullptr;                 // [uqn, qrp]
  void* w_ukT = nullptr;                // [heads][kv_rank, dimp]
  void* w_uv = nullptr;                 // [heads][vdim, kvp]
  int qrp = 0, uqn = 0, dimp = 0, kvp = 0, Dk = 0, ldpool = 0, ldqa = 0, ldol = 0;
  void* pool = nullptr;                 // [slots, ldpool]: [normed latent | rotated key part] per token (own layers)
  const float* rot = nullptr;
};

struct nvc_latent_body : nvc_body_base {
  float *lat_qf = nullptr, *lat_hv = nullptr;
  void *lat_cq = nullptr, *lat_qn = nullptr, *lat_qabs = nullptr, *lat_olat = nullptr;
  size_t lat_qrp = 0, lat_uqn = 0, lat_qn_cols = 0, lat_qa = 0, lat_ol = 0, lat_hv_cols = 0;

  // sizes, weights and pool of one layer; off = first free column of its projection row.  *columns = columns the layer reads there.
  int latent_init(nvc_runner* r, const nvc_latent_attn_spec& a, const std::string& p, size_t slots, int off, nvc_latent_weights& w, int* columns,
                  int64_t* weights) {
    const bool own = a.kv_from < 0;
    int rc;
    w.Dk = a.kv_rank + a.rot_dim;
    NVC_REQUIRE(r->ctx, w.Dk <= 512, NVC_ESHAPE, "kv_rank + rot_dim above 512");
    w.dq_off = off;
    w.kv_off = off + a.q_rank;
    *columns = a.q_rank + (own ? w.Dk : 0);
    w.qrp = pad64(a.q_rank);
    w.uqn = pad64(a.heads * (a.dim + a.rot_dim));
    w.dimp = pad8(a.dim);
    w.kvp = pad8(a.kv_rank);
    w.ldpool = pad8(w.Dk);
    w.ldqa = pad8(a.heads * w.Dk);
    w.ldol = pad8(a.heads * w.Dk);          // room for value columns as wide as the key (the tcgen05 route)
    if ((rc = zalloc(r, &w.dq_norm, a.q_rank * 4)) || (rc = zalloc(r, &w.w_uq, (size_t)w.uqn * w.qrp * esz)) ||
        (rc = zalloc(r, &w.w_ukT, (size_t)a.heads * a.kv_rank * w.dimp * esz)) || (rc = zalloc(r, &w.w_uv, (size_t)a.heads * a.vdim * w.kvp * esz)))
      return rc;
    for (const char* n : {"mix.dq", "mix.dq.norm", "mix.uq", "mix.uk", "mix.uv"}) want[p + n] = false;
    if (own) {
      if ((rc = zalloc(r, &w.dkv_norm, a.kv_rank * 4)) || (rc = zalloc(r, &w.pool, slots * w.ldpool * esz))) return rc;
      want[p + "mix.dkv"] = false;
      want[p + "mix.dkv.norm"] = false;
    }
    if (a.sink) {
      if ((rc = zalloc(r, &w.sink, a.heads * 4))) return rc;
      want[p + "mix.sink"] = false;
    }
    if ((rc = rotary_table(r, a.rot, &w.rot))) return rc;
    *weights += (int64_t)a.heads * (a.dim + a.rot_dim) * a.q_rank + (int64_t)a.heads * (a.dim + a.vdim) * a.kv_rank;
    lat_qrp = std::max(lat_qrp, (size_t)w.qrp);
    lat_uqn = std::max(lat_uqn, (size_t)w.uqn);
    lat_qn_cols = std::max(lat_qn_cols, (size_t)a.heads * w.dimp);
    lat_qa = std::max(lat_qa, (size_t)w.ldqa);
    lat_ol = std::max(lat_ol, (size_t)w.ldol);
    if (a.gate) lat_hv_cols = std::max(lat_hv_cols, (size_t)a.heads * a.vdim);
    return NVC_OK;
  }

  // activations for steps of up to T rows, once every layer is known (zeroed: padding columns are never written)
  int latent_alloc(nvc_runner* r, size_t T) {
    int rc;
    if (lat_uqn && ((rc = zalloc(r, &lat_cq, T * lat_qrp * esz)) || (rc = zalloc(r, &lat_qf, T * lat_uqn * 4)) || (rc = zalloc(r, &lat_qn, T * lat_qn_cols * esz)) ||
                    (rc = zalloc(r, &lat_qabs, T * lat_qa * esz)) || (rc = zalloc(r, &lat_olat, T * lat_ol * esz))))
      return rc;
    return lat_hv_cols ? zalloc(r, &lat_hv, T * lat_hv_cols * 4) : NVC_OK;
  }

  // one tensor of a latent layer (sub = its name behind the layer's prefix); *taken = false when it is none of the mixer's own.
  // in_rows(off, rows) writes rows of the fused input projection, bad() reports a shape.
  template <typename InRows, typename Bad>
  int latent_load(nvc_runner* r, const nvc_latent_attn_spec& a, nvc_latent_weights& w, const std::string& sub, const std::vector<float>& v, int64_t d0, int64_t d1,
                  InRows&& in_rows, Bad&& bad, bool* taken) {
    int rc = NVC_OK;
    *taken = true;
    auto vec = [&](float* dst, size_t len) { return v.size() == len ? put_f32(r, dst, v.data(), len) : bad(); };
    auto shape_is = [&](int64_t x, int64_t y) { return d0 == x && d1 == y; };
    if (sub == "mix.dq") return in_rows(w.dq_off, a.q_rank);
    if (sub == "mix.dkv") return in_rows(w.kv_off, w.Dk);
    if (sub == "mix.dq.norm") return vec(w.dq_norm, a.q_rank);
    if (sub == "mix.dkv.norm") return vec(w.dkv_norm, a.kv_rank);
    if (sub == "mix.sink") return vec(w.sink, a.heads);
    if (sub == "mix.uq") {
      if (!shape_is(a.heads * (a.dim + a.rot_dim), a.q_rank)) return bad();
      return put_matrix(r, w.w_uq, w.qrp, 0, 0, v.data(), a.heads * (a.dim + a.rot_dim), a.q_rank, a.q_rank, 1);
    }
    if (sub == "mix.uk") {
      // [heads * dim, kv_rank] -> per head the transposed block [kv_rank, dimp]: q' = W_uk,h^T q
      if (!shape_is(a.heads * a.dim, a.kv_rank)) return bad();
      for (int hh = 0; hh < a.heads && rc == NVC_OK; ++hh)
        rc = put_matrix(r, reinterpret_cast<uint8_t*>(w.w_ukT) + (size_t)hh * a.kv_rank * w.dimp * esz, w.dimp, 0, 0,
                        v.data() + (size_t)hh * a.dim * a.kv_rank, a.kv_rank, a.dim, 1, a.kv_rank);
      return rc;
    }
    if (sub == "mix.uv") {
      if (!shape_is(a.heads * a.vdim, a.kv_rank)) return bad();
      for (int hh = 0; hh < a.heads && rc == NVC_OK; ++hh)
        rc = put_matrix(r, reinterpret_cast<uint8_t*>(w.w_uv) + (size_t)hh * a.vdim * w.kvp * esz, w.kvp, 0, 0,
                        v.data() + (size_t)hh * a.vdim * a.kv_rank, a.vdim, a.kv_rank, a.kv_rank, 1);
      return rc;
    }
    *taken = false;
    return NVC_OK;
  }


  // attention over a pool of shared rows, keys and values at once: one-token sequences of a mixed step come first in the batch and keep
  // the decode path of the wide kernel, the portions behind them take the tcgen05 kernel when `flash`
  int shared_attention(nvc_runner* r, const nvc_step_shape& s, const nvc_attn_spec& sp, bool flash, const void* q, int ldq, const void* pool, int ldpool,
                       void* out, int ldo) {
    nvc_ctx* ctx = r->ctx;
    void* st = r->stream;
    const int bs = r->opt.kvcache_block_size, cap = r->max_blocks_cap;
    if (!flash)
      return nvc_attn_paged_wide(ctx, q, ldq, pool, ldpool, pool, ldpool, r->d_bt, cap, r->d_ctx, s.decode ? nullptr : r->d_cu, s.B, s.N,
                                 s.decode ? 1 : s.max_seqlen, bs, &sp, out, ldo, dt, st);
    const int nd = s.num_decode;
    int rc;
    if (nd > 0 && (rc = nvc_attn_paged_wide(ctx, q, ldq, pool, ldpool, pool, ldpool, r->d_bt, cap, r->d_ctx, nullptr, nd, nd, 1, bs, &sp, out, ldo, dt, st)))
      return rc;
    nvc_attn_spec sq = sp;
    if (sq.gate) sq.gate += (size_t)nd * sq.ldg;
    return nvc_prefill_attn_shared(ctx, reinterpret_cast<const nvc_bf16*>(q) + (size_t)nd * ldq, ldq, reinterpret_cast<const nvc_bf16*>(pool),
                                   r->d_bt + (size_t)nd * cap, cap, r->d_ctx + nd, nd ? r->d_cu2 : r->d_cu, s.B - nd, s.N - nd, s.max_chunk, bs,
                                   r->opt.num_kvcache_blocks, &sq, reinterpret_cast<nvc_bf16*>(out) + (size_t)nd * ldo, ldo, st);
  }

  // the mixer behind the input projection `proj` (row stride np) up to the input of the output projection, ao [N, owp].  source = the layer
  // whose pool is read (w itself, or the one named by kv_from); gate: fp32 columns [heads * vdim] of a row (a.gate)
  int latent_run(nvc_runner* r, const nvc_step_shape& s, const nvc_latent_attn_spec& a, const nvc_latent_weights& w, const nvc_latent_weights& source, float eps,
                 const float* proj, int np, const float* gate, void* ao, int owp) {
    nvc_ctx* ctx = r->ctx;
    void* st = r->stream;
    const int N = s.N;
    const bool own = a.kv_from < 0;
    int rc;
    // the kernel takes the query latent's columns from the row's start and the key latent's offset relative to it
    if ((rc = nvc_latent_norm_store_rot(ctx, proj + w.dq_off, np, a.q_rank, w.kv_off - w.dq_off, own ? a.kv_rank : 0, w.dq_norm, w.dkv_norm, eps, lat_cq, w.qrp,
                                        own ? w.pool : nullptr, w.ldpool, r->d_slots, a.rot_dim, a.rot.dims, a.rot_half ? 1 : 0, w.rot, r->d_pos, dt, N, st)))
      return rc;
    mark(r, "latent_norm_store");
    if ((rc = linear(r, lat_cq, w.qrp, w.w_uq, lat_qf, w.uqn, NVC_DT_F32, N, w.uqn, w.qrp))) return rc;
    mark(r, "gemm_uq");
    const int hd = a.heads * w.dimp;
    if ((rc = nvc_head_split_rot(ctx, lat_qf, w.uqn, a.heads, a.dim, a.rot_dim, a.rot.dims, a.rot_half ? 1 : 0, w.rot, r->d_pos, lat_qn, hd, w.dimp, lat_qabs,
                                 w.ldqa, w.Dk, a.kv_rank, dt, N, st)))
      return rc;
    mark(r, "q_split_rot");
    if ((rc = nvc_linear(ctx, lat_qn, hd, w.dimp, w.w_ukT, w.dimp, (int64_t)a.kv_rank * w.dimp, lat_qabs, w.ldqa, w.Dk, dt, dt, N, a.kv_rank, w.dimp, a.heads,
                         NVC_ACT_NONE, st)))
      return rc;
    mark(r, "absorb_uk");
    // key = value = the whole row on the tcgen05 route: the value columns behind the latent come out as a weighted sum of rotated key
    // parts, which the value up-projection never reads (all sequences of the step then share that output layout)
    const bool flash = w.Dk == 128 && w.ldpool == 128 && flash_step(r, s);
    nvc_attn_spec sp{};
    sp.heads = a.heads; sp.kv_heads = 1; sp.dim = w.Dk; sp.vdim = flash ? w.Dk : a.kv_rank;
    sp.scale = a.scale;
    sp.window = a.window;
    sp.sink = a.sink ? w.sink : nullptr;
    sp.out_scale = 1.f;
    if ((rc = shared_attention(r, s, sp, flash, lat_qabs, w.ldqa, source.pool, w.ldpool, lat_olat, w.ldol))) return rc;
    mark(r, "attention");
    const int ohs = sp.vdim, vw = a.heads * a.vdim, K = ohs % 8 == 0 ? w.kvp : a.kv_rank;      // ohs: numbers per head in lat_olat
    if (!a.gate) {
      rc = nvc_linear(ctx, lat_olat, w.ldol, ohs, w.w_uv, w.kvp, (int64_t)a.vdim * w.kvp, ao, owp, a.vdim, dt, dt, N, a.vdim, K, a.heads, NVC_ACT_NONE, st);
      mark(r, "absorb_uv");
      return rc;
    }
    if ((rc = nvc_linear(ctx, lat_olat, w.ldol, ohs, w.w_uv, w.kvp, (int64_t)a.vdim * w.kvp, lat_hv, vw, a.vdim, dt, NVC_DT_F32, N, a.vdim, K, a.heads,
                         NVC_ACT_NONE, st)))
      return rc;
    mark(r, "absorb_uv");
    if ((rc = nvc_head_gate(ctx, lat_hv, vw, gate, np, ao, owp, dt, a.heads, a.vdim, 0, eps, NVC_GATE_SIGMOID, 1.f, N, st))) return rc;
    mark(r, "head_gate");
    return NVC_OK;
  }
};

}  // namespace
