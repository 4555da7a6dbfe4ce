// Decode rows of nvc_attn_paged_wide over SHARED rows (bf16; the values are the leading numbers of the key rows, 64 or 128 numbers each):
// one query token per sequence, 16 (token, head) rows at most per CTA.  Included by attn_wide_mma.cuh only.
//
// The products are taken transposed, with the 16 cached tokens of a tile as the M dimension and the query heads as N: a key / value head
// with up to 8 query heads fills one n-tile of 8 instead of half of a 16-row M - half the MMAs and half the exponentials of the row-major
// form (attn_wide_mma_kernel), and a third of its registers, so that four CTAs stay resident per SM.
//   S^T = K Q^T:     A = the tile (ldmatrix), B = the query heads (registers for the whole launch)
//   P^T:             in accumulator layout, turned into a B operand by movmatrix (no shared-memory round trip)
//   O^T += V^T P^T:  A = the same tile (ldmatrix.trans)
// Warp w of a CTA owns the 16-token tiles w, w + 4, ... (of the CTA's share of the keys when a cluster splits them) in a private
// cp.async ring of three tiles; a tile lies in one page, whose table entry is fetched one tile ahead.  Tiles that cannot hold this
// step's own rows are requested before the launch dependency is waited for.  Softmax keeps a running maximum that moves only when
// some score outgrows it by 2^8 (exact after the final division); sigmoid weights need none.
#pragma once

namespace widemma {

constexpr int kSdTok = 16;                            // tokens per warp tile
template <int DK> constexpr int shared_decode_smem() {
  constexpr int ring = kWarps * kStages * (kSdTok * DK * 2 + kSdTok * 4);
  constexpr int merge = (2 * kWarps * 16 + 2 * 16 + kWarps * 16 * DK) * 4;
  return ring > merge ? ring : merge;
}

__device__ __forceinline__ uint32_t movmatrix_trans(uint32_t x) {
  uint32_t y;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
  return y;
}
__device__ __forceinline__ float ld_shared_f(uint32_t addr) {
  float v;
  asm volatile("ld.shared.f32 %0, [%1];" : "=f"(v) : "r"(addr));
  return v;
}

// NR: n-tiles of 8 query heads (1 or 2)
template <int DK, int NR, bool kSig>
__global__ void __launch_bounds__(kWarps * 32, 4) attn_shared_decode_kernel(const Args a) {
  constexpr int RB = DK * 2, KS = DK / 16, NCK = DK / 8, RPI = 32 / NCK, ITS = kSdTok / RPI;
  constexpr int kTile = kSdTok * RB;
  constexpr float kLazy = 8.0f;                       // the running maximum moves when a score outgrows it by 2^8
  extern __shared__ __align__(1024) uint8_t smem[];
  pdl_trigger();
  const int b = blockIdx.y, g = blockIdx.z;
  const int hg = a.heads / a.kv_heads;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int quad = lane >> 2, tq = lane & 3;
  const int split = (int)blockIdx.x % a.splits;
  const int r0 = (int)blockIdx.x / a.splits * 16;     // first head of the group this CTA takes
  const int nrows = min(16, hg - r0);
  const int pos = __ldg(a.context_lens + b) - 1;
  const int lo = first_visible(pos, a.window, a.chunk);
  const int32_t* bt = a.block_tables + (int64_t)b * a.bt_stride;
  // ---- this warp's tiles
  const int stride = kWarps * kSdTok * a.splits;
  const int first = lo / kSdTok * kSdTok + (split * kWarps + warp) * kSdTok;
  const int n_tiles = first <= pos ? (pos - first) / stride + 1 : 0;
  const uint32_t ring = smem_u32(smem) + warp * (kStages * kTile);
  const uint32_t sring = smem_u32(smem) + kWarps * kStages * kTile + warp * (kStages * kSdTok * 4);
  const int srow = lane / NCK, schunk = lane % NCK;   // a warp-wide copy brings RPI rows
  const int64_t pitch = (int64_t)a.ldk * 2;
  const uint8_t* src0 = reinterpret_cast<const uint8_t*>(a.k_cache + (int64_t)g * DK) + srow * pitch + schunk * 16;
  const uint32_t dst0 = srow * RB + ((schunk ^ srow) << 4);
  auto slot_of = [&](int i) -> int64_t {              // first row of tile i in the pool
    const int t = first + i * stride, blk = t / a.block_size;
    return (int64_t)__ldg(bt + blk) * a.block_size + (t - blk * a.block_size);
  };
  auto load = [&](int i, int64_t slot) {
    const int st_i = i % kStages;
    const uint32_t d = ring + st_i * kTile + dst0;
    const uint8_t* s = src0 + slot * pitch;
    const int nvalid = pos - (first + i * stride) + 1;            // rows of the tile inside the context
    if (nvalid >= kSdTok) {
#pragma unroll
      for (int it = 0; it < ITS; ++it) cp_async16((d ^ ((it * RPI & 7) << 4)) + it * RPI * RB, s + it * RPI * pitch, 16u);
    } else {
#pragma unroll
      for (int it = 0; it < ITS; ++it) {
        const bool ok = it * RPI + srow < nvalid;
        cp_async16((d ^ ((it * RPI & 7) << 4)) + it * RPI * RB, ok ? s + it * RPI * pitch : s - srow * pitch, ok ? 16u : 0u);
      }
    }
    if (a.key_scale && lane < kSdTok) {
      const bool ok = lane < nvalid;
      cp_async4(sring + (st_i * kSdTok + lane) * 4, a.key_scale + slot + (ok ? lane : 0), ok ? 4u : 0u);
    }
  };
  // only the tile of position `pos` holds a row of this step: the others may fly before the dependency is resolved
  int64_t next_slot = n_tiles > 0 ? slot_of(0) : 0;
  bool waited = false;
#pragma unroll
  for (int p = 0; p < kStages - 1; ++p) {
    if (p < n_tiles) {
      if (!waited && first + p * stride + kSdTok > pos) { pdl_wait(); waited = true; }
      load(p, next_slot);
      if (p + 1 < n_tiles) next_slot = slot_of(p + 1);
    }
    cp_async_commit();
  }
  if (!waited) pdl_wait();
  // ---- the query heads as B operands (heads past the end are zero)
  uint32_t qb[NR][KS][2];
  float bias[NR][2];
#pragma unroll
  for (int t = 0; t < NR; ++t) {
    const int h = t * 8 + quad;
    const nvc_bf16* qr = a.q + (int64_t)b * a.ldq + (int64_t)(g * hg + r0 + min(h, nrows - 1)) * DK;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      const bool in = h < nrows;
      qb[t][ks][0] = in ? *reinterpret_cast<const uint32_t*>(qr + ks * 16 + 2 * tq) : 0u;
      qb[t][ks][1] = in ? *reinterpret_cast<const uint32_t*>(qr + ks * 16 + 2 * tq + 8) : 0u;
    }
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      const int hc = t * 8 + 2 * tq + c;
      bias[t][c] = kSig && a.bias && hc < nrows ? __ldg(a.bias + g * hg + r0 + hc) * kLog2e : 0.f;
    }
  }
  const int mt_n = a.dv >> 4;
  float o[KS][NR][4];                                 // O^T: 16 numbers x 8 heads per tile
#pragma unroll
  for (int mt = 0; mt < KS; ++mt)
#pragma unroll
    for (int t = 0; t < NR; ++t) o[mt][t][0] = o[mt][t][1] = o[mt][t][2] = o[mt][t][3] = 0.f;
  float m[NR][2], l[NR][2];
#pragma unroll
  for (int t = 0; t < NR; ++t) { m[t][0] = m[t][1] = -INFINITY; l[t][0] = l[t][1] = 0.f; }
  // ldmatrix lanes: rows 0-7 | 8-15 of the tile for S (chunk + 1 for lanes 16-31), chunk | chunk + 1 for V (rows + 8 for lanes 16-31)
  const int rs = (lane & 7) + ((lane >> 3) & 1) * 8, rv = (lane & 7) + (lane >> 4) * 8;
  const uint32_t ls = rs * RB + (((lane >> 4) ^ (lane & 7)) << 4), lv = rv * RB + ((((lane >> 3) & 1) ^ (lane & 7)) << 4);

  for (int i = 0; i < n_tiles; ++i) {
    if (i + kStages - 1 < n_tiles) {
      load(i + kStages - 1, next_slot);
      if (i + kStages < n_tiles) next_slot = slot_of(i + kStages);
    }
    cp_async_commit();
    cp_async_wait<kStages - 1>();
    __syncwarp();
    const uint32_t st = ring + (i % kStages) * kTile;
    float s[NR][4];
#pragma unroll
    for (int t = 0; t < NR; ++t) s[t][0] = s[t][1] = s[t][2] = s[t][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      uint32_t f[4];
      ldmatrix_x4((st + ls) ^ (ks << 5), f[0], f[1], f[2], f[3]);
#pragma unroll
      for (int t = 0; t < NR; ++t) mma_bf16(s[t], f, qb[t][ks][0], qb[t][ks][1]);
    }
    // s[t][0..1]: token quad, heads 8 t + 2 tq + {0, 1};  s[t][2..3]: token quad + 8
    float f0 = a.scale_log2e, f1 = a.scale_log2e;
    if (a.key_scale) {
      const uint32_t sc = sring + ((i % kStages) * kSdTok + quad) * 4;
      f0 *= ld_shared_f(sc);
      f1 *= ld_shared_f(sc + 32);
    }
    const int t0 = first + i * stride;
    const bool edge = t0 < lo || t0 + kSdTok - 1 > pos;
    const bool v0 = t0 + quad >= lo && t0 + quad <= pos, v1 = t0 + quad + 8 >= lo && t0 + quad + 8 <= pos;
    uint32_t pb[NR][2];
    if constexpr (kSig) {
#pragma unroll
      for (int t = 0; t < NR; ++t) {
        float p0 = sigmoid_exp2(fmaf(s[t][0], f0, bias[t][0])), p1 = sigmoid_exp2(fmaf(s[t][1], f0, bias[t][1]));
        float p2 = sigmoid_exp2(fmaf(s[t][2], f1, bias[t][0])), p3 = sigmoid_exp2(fmaf(s[t][3], f1, bias[t][1]));
        if (edge) {
          if (!v0) p0 = p1 = 0.f;
          if (!v1) p2 = p3 = 0.f;
        }
        pb[t][0] = movmatrix_trans(pack_bf16(p0, p1));
        pb[t][1] = movmatrix_trans(pack_bf16(p2, p3));
      }
    } else {
      bool grow = false;
#pragma unroll
      for (int t = 0; t < NR; ++t) {
        s[t][0] = !edge || v0 ? s[t][0] * f0 : -INFINITY;
        s[t][1] = !edge || v0 ? s[t][1] * f0 : -INFINITY;
        s[t][2] = !edge || v1 ? s[t][2] * f1 : -INFINITY;
        s[t][3] = !edge || v1 ? s[t][3] * f1 : -INFINITY;
        grow = grow || fmaxf(s[t][0], s[t][2]) > m[t][0] + kLazy || fmaxf(s[t][1], s[t][3]) > m[t][1] + kLazy;
      }
      if (__any_sync(0xffffffffu, grow)) {
#pragma unroll
        for (int t = 0; t < NR; ++t) {
          float al[2];
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            float mx = fmaxf(s[t][c], s[t][2 + c]);
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 4));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 8));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 16));
            mx = fmaxf(mx, m[t][c]);
            al[c] = mx == -INFINITY ? 1.f : fast_exp2(m[t][c] - mx);
            m[t][c] = mx;
            l[t][c] *= al[c];
          }
#pragma unroll
          for (int mt = 0; mt < KS; ++mt) {
            o[mt][t][0] *= al[0]; o[mt][t][1] *= al[1];
            o[mt][t][2] *= al[0]; o[mt][t][3] *= al[1];
          }
        }
      }
#pragma unroll
      for (int t = 0; t < NR; ++t) {
        const float m0 = m[t][0] == -INFINITY ? 0.f : m[t][0], m1 = m[t][1] == -INFINITY ? 0.f : m[t][1];
        const float p0 = fast_exp2(s[t][0] - m0), p1 = fast_exp2(s[t][1] - m1), p2 = fast_exp2(s[t][2] - m0), p3 = fast_exp2(s[t][3] - m1);
        l[t][0] += p0 + p2;
        l[t][1] += p1 + p3;
        pb[t][0] = movmatrix_trans(pack_bf16(p0, p1));
        pb[t][1] = movmatrix_trans(pack_bf16(p2, p3));
      }
    }
#pragma unroll
    for (int mt = 0; mt < KS; ++mt) {
      if (mt < mt_n) {
        uint32_t f[4];
        ldmatrix_x4_trans((st + lv) ^ (mt << 5), f[0], f[1], f[2], f[3]);
#pragma unroll
        for (int t = 0; t < NR; ++t) mma_bf16(o[mt][t], f, pb[t][0], pb[t][1]);
      }
    }
    __syncwarp();
  }
  cp_async_wait<0>();
  __syncthreads();                                    // the rings are dead now: partial results take their place
  float* sm_m = reinterpret_cast<float*>(smem);       // [kWarps][16]
  float* sm_l = sm_m + kWarps * 16;
  float* cta_ml = sm_l + kWarps * 16;                 // [2][16]
  float* sm_o = cta_ml + 32;                          // [kWarps][16][DK]
#pragma unroll
  for (int t = 0; t < NR; ++t) {
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      float s = l[t][c];
      s += __shfl_xor_sync(0xffffffffu, s, 4);
      s += __shfl_xor_sync(0xffffffffu, s, 8);
      s += __shfl_xor_sync(0xffffffffu, s, 16);
      const int row = t * 8 + 2 * tq + c;
      if (quad == 0) { sm_m[warp * 16 + row] = m[t][c]; sm_l[warp * 16 + row] = s; }
#pragma unroll
      for (int mt = 0; mt < KS; ++mt) {
        if (mt < mt_n) {
          sm_o[(warp * 16 + row) * DK + mt * 16 + quad] = o[mt][t][c];
          sm_o[(warp * 16 + row) * DK + mt * 16 + quad + 8] = o[mt][t][2 + c];
        }
      }
    }
  }
  __syncthreads();
  merge_store<DK, kSig>(a, sm_m, sm_l, cta_ml, sm_o, nrows, r0, hg, g, b);
}

}  // namespace widemma

namespace {

// without cu_seqlens every sequence has one row
inline bool attn_shared_decode_takes(const nvc_attn_spec& s, bool shared, const int32_t* cu_seqlens, int block_size) {
  return !cu_seqlens && shared && (s.dim == 64 || s.dim == 128) && block_size % 16 == 0 && s.softcap == 0.f;
}

template <int DK, int NR, bool kSig>
inline int attn_shared_decode_launch_t(nvc_ctx* ctx, const widemma::Args& a, dim3 grid, cudaStream_t stream) {
  constexpr int smem = widemma::shared_decode_smem<DK>();
  static bool attr_set = false;
  if (!attr_set) {
    NVC_CUDA_CHECK(ctx, cudaFuncSetAttribute(widemma::attn_shared_decode_kernel<DK, NR, kSig>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    NVC_CUDA_CHECK(ctx, cudaFuncSetAttribute(widemma::attn_shared_decode_kernel<DK, NR, kSig>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
    attr_set = true;
  }
  NVC_CUDA_CHECK(ctx, nvc_launch_cluster(ctx, widemma::attn_shared_decode_kernel<DK, NR, kSig>, grid, dim3(widemma::kWarps * 32), (size_t)smem, stream,
                                         a.splits, a));
  ctx->launches++;
  return NVC_OK;
}

inline int attn_shared_decode_launch(nvc_ctx* ctx, const widemma::Args& a, int hg, dim3 grid, bool sig, cudaStream_t stream) {
  const bool one = hg <= 8, wide = a.dk == 128;
  if (sig)
    return wide ? (one ? attn_shared_decode_launch_t<128, 1, true>(ctx, a, grid, stream) : attn_shared_decode_launch_t<128, 2, true>(ctx, a, grid, stream))
                : (one ? attn_shared_decode_launch_t<64, 1, true>(ctx, a, grid, stream) : attn_shared_decode_launch_t<64, 2, true>(ctx, a, grid, stream));
  return wide ? (one ? attn_shared_decode_launch_t<128, 1, false>(ctx, a, grid, stream) : attn_shared_decode_launch_t<128, 2, false>(ctx, a, grid, stream))
              : (one ? attn_shared_decode_launch_t<64, 1, false>(ctx, a, grid, stream) : attn_shared_decode_launch_t<64, 2, false>(ctx, a, grid, stream));
}

}  // namespace
