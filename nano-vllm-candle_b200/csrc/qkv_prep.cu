// nvc_qkv_prep: everything between the fused q / k / v projection of a mixer and its attention or recurrence, in one pass
// over the fp32 projection rows:
//   + bias                                   (optional)
//   silu                                     (optional, on q, k and v)
//   per-head RMS norm of q and k             (optional; one weight vector of `dim` numbers shared by the heads, or no weight)
//   rotary positions on the first rot_dims numbers of every q / k head, pairs (2i, 2i + 1) or (i, i + rot_dims / 2),
//                                            angles from a table of (cos, sin) per position
//   k *= k_scale                             (after the rotation)
//   value blending                           v <- (1 - lambda) v + lambda v_first, or v_first <- v in the layer that provides it
//   v *= v_scale                             (a constant weight of the mixer, so that every attention kernel can leave it out)
//   stores                                   q to its buffer; k and v to rows of a paged cache (slot mapping) or to plain rows
// One warp per (token, head) of q, k or v; a head is staged in shared memory so that any pairing reads its partner.  The purely
// element-wise case (bias and silu only, plain fp32 rows out) runs a flat kernel with 16-byte accesses instead.  With a short causal
// convolution behind the bias, or norms that span the whole query / key projection, one CTA takes a whole token (prep_token_kernel).
#include "typed.cuh"

#include <algorithm>
#include <cmath>

namespace {

struct PrepArgs {
  nvc_qkv_prep p;
  int N;
};

template <typename TQ, typename TKV>
__global__ void qkv_prep_kernel(const PrepArgs a) {
  extern __shared__ float stage[];
  pdl_trigger();
  pdl_wait();
  const nvc_qkv_prep& p = a.p;
  const int warps = blockDim.x >> 5, wid = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int units = p.q_heads + 2 * p.kv_heads;
  const int64_t u = (int64_t)blockIdx.x * warps + wid;
  if (u >= (int64_t)a.N * units) return;
  const int n = (int)(u / units), uu = (int)(u % units);
  const int wmax = p.dim > p.vdim ? p.dim : p.vdim;
  float* x = stage + (size_t)wid * wmax;
  const float* in = p.in + (int64_t)n * p.ldi;
  if (uu >= p.q_heads + p.kv_heads) {
    // ---- a value head
    const int h = uu - p.q_heads - p.kv_heads;
    const int col = p.v_off + h * p.vdim;
    const int64_t orow = p.slot_mapping ? p.slot_mapping[n] : n;
    const float lam = p.blend == NVC_BLEND_MIX ? __ldg(p.lambda) : 0.f;
    for (int j = lane; j < p.vdim; j += 32) {
      float v = in[col + j] + (p.bias ? __ldg(p.bias + col + j) : 0.f);
      if (p.act == NVC_PREP_ACT_SILU) v = v * sigmoid_f32(v);
      if (p.blend == NVC_BLEND_PROVIDE) p.v_first[(int64_t)n * p.ldvf + h * p.vdim + j] = v;
      else if (p.blend == NVC_BLEND_MIX) v = (1.0f - lam) * v + lam * p.v_first[(int64_t)n * p.ldvf + h * p.vdim + j];
      v *= p.v_scale;
      if (orow >= 0) st_f(reinterpret_cast<TKV*>(p.v_out) + orow * p.ldv + h * p.vdim + j, v);
    }
    return;
  }
  const bool is_q = uu < p.q_heads;
  const int h = is_q ? uu : uu - p.q_heads;
  const int col = (is_q ? p.q_off : p.k_off) + h * p.dim;
  const int64_t orow = is_q ? n : (p.slot_mapping ? p.slot_mapping[n] : n);
  if (orow < 0) return;
  float ss = 0.f;
  for (int j = lane; j < p.dim; j += 32) {
    float v = in[col + j] + (p.bias ? __ldg(p.bias + col + j) : 0.f);
    if (p.act == NVC_PREP_ACT_SILU) v = v * sigmoid_f32(v);
    x[j] = v;
    ss += v * v;
  }
  const float* nw = is_q ? p.q_norm : p.k_norm;
  float r = 1.f;
  if (nw || p.unit_norm) {
    ss = warp_sum(ss);
    r = 1.0f / sqrtf(ss / (float)p.dim + p.eps);
  }
  __syncwarp();
  const int half = p.rot_dims >> 1;
  const float2* tab = reinterpret_cast<const float2*>(p.rot_table) + (int64_t)(p.rot_dims ? p.positions[n] : 0) * half;
  const float post = is_q ? 1.f : p.k_scale;
  for (int j = lane; j < p.dim; j += 32) {
    float y = x[j] * r * (nw ? __ldg(nw + j) : 1.f);
    if (j < p.rot_dims) {
      int i, partner;
      float sign;
      if (p.rot_half) { i = j < half ? j : j - half; partner = j < half ? j + half : j - half; sign = j < half ? -1.f : 1.f; }
      else { i = j >> 1; partner = j ^ 1; sign = (j & 1) ? 1.f : -1.f; }
      const float2 cs = __ldg(tab + i);
      const float z = x[partner] * r * (nw ? __ldg(nw + partner) : 1.f);
      y = y * cs.x + sign * z * cs.y;
    }
    y *= post;
    if (is_q) st_f(reinterpret_cast<TQ*>(p.q_out) + orow * p.ldq + h * p.dim + j, y);
    else st_f(reinterpret_cast<TKV*>(p.k_out) + orow * p.ldk + h * p.dim + j, y);
  }
}


// The element-wise case (no norm, no rotation, no blending, no scale, plain fp32 rows out): q, k, v = act(in + bias), four numbers per
// thread.  CTA = (token, block of 256 x 4 columns of [q | k | v]).
__global__ void __launch_bounds__(256) prep_flat_kernel(const PrepArgs a) {
  pdl_trigger();
  pdl_wait();
  const nvc_qkv_prep& p = a.p;
  const int qw = p.q_heads * p.dim, kw = p.kv_heads * p.dim, vw = p.kv_heads * p.vdim;
  const int64_t n = blockIdx.x;
  const int j = 4 * (blockIdx.y * blockDim.x + threadIdx.x);          // column of [q | k | v]
  if (j >= qw + kw + vw) return;
  int col;
  float* out;
  if (j < qw) { col = p.q_off + j; out = reinterpret_cast<float*>(p.q_out) + n * p.ldq + j; }
  else if (j < qw + kw) { col = p.k_off + j - qw; out = reinterpret_cast<float*>(p.k_out) + n * p.ldk + j - qw; }
  else { col = p.v_off + j - qw - kw; out = reinterpret_cast<float*>(p.v_out) + n * p.ldv + j - qw - kw; }
  float4 v = *reinterpret_cast<const float4*>(p.in + n * p.ldi + col);
  if (p.bias) {
    const float4 b = *reinterpret_cast<const float4*>(p.bias + col);
    v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
  }
  if (p.act == NVC_PREP_ACT_SILU) { v.x *= sigmoid_f32(v.x); v.y *= sigmoid_f32(v.y); v.z *= sigmoid_f32(v.z); v.w *= sigmoid_f32(v.w); }
  *reinterpret_cast<float4*>(out) = v;
}

// four neighbouring numbers in the storage format with one store
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
  uint2 u;
  u.x = pack_bf16(v.x, v.y);
  u.y = pack_bf16(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = u;
}

__device__ __forceinline__ int prep_find_seq(const int32_t* cu, int B, int row) {
  int lo = 0, hi = B - 1;      // largest b with cu[b] <= row
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= row) lo = mid; else hi = mid - 1;
  }
  return lo;
}

// One CTA per token: bias, short causal convolution, activation (the whole row [q | k | v] waits in shared memory), the norms over the
// whole query and key projection - or none - then rotation and stores.  P: numbers per access (4: every width, offset and stride is a
// multiple of 4 and the pointers are 16-byte aligned).  TAPS: the convolution's taps when they are 2 .. 4 (all inputs of a channel are in
// flight at once), 0: any number of them, or no convolution.
template <typename TQ, typename TKV, int P, int TAPS>
__global__ void __launch_bounds__(1024) prep_token_kernel(const PrepArgs a, const nvc_short_conv cv) {
  extern __shared__ __align__(16) float row[];          // [qw + kw + vw]
  __shared__ float part[2][32];
  __shared__ int s_r0, s_fresh, s_slot;
  pdl_trigger();
  const nvc_qkv_prep& p = a.p;
  const int qw = p.q_heads * p.dim, kw = p.kv_heads * p.dim, vw = p.kv_heads * p.vdim, C = qw + kw + vw;
  const int64_t n = blockIdx.x;
  if (cv.w && threadIdx.x == 0) {
    int b = (int)n, r0 = (int)n;
    if (cv.cu_seqlens) {
      b = prep_find_seq(cv.cu_seqlens, cv.B, (int)n);
      r0 = cv.cu_seqlens[b];
    }
    s_r0 = r0;
    s_fresh = p.positions[r0] == 0;
    s_slot = cv.state_slots[b];
  }
  const int64_t orow = p.slot_mapping ? p.slot_mapping[n] : n;
  pdl_wait();
  __syncthreads();
  const int step = P * blockDim.x;
  float sq = 0.f, sk = 0.f;
  for (int c = P * threadIdx.x; c < C; c += step) {
    const int col = c < qw ? p.q_off + c : (c < qw + kw ? p.k_off + c - qw : p.v_off + c - qw - kw);
    float b[P], y[P] = {};
    if constexpr (P == 4) {
      const float4 t = p.bias ? *reinterpret_cast<const float4*>(p.bias + col) : make_float4(0.f, 0.f, 0.f, 0.f);
      b[0] = t.x; b[1] = t.y; b[2] = t.z; b[3] = t.w;
    } else {
      b[0] = p.bias ? __ldg(p.bias + col) : 0.f;
    }
    if (TAPS > 0 || cv.w) {
      const int taps = TAPS > 0 ? TAPS : cv.taps, keep = taps - 1, t = (int)n - s_r0;
      float* st = cv.state + (int64_t)s_slot * keep * C + c;
      const bool shift = cv.cu_seqlens == nullptr;      // one row per sequence: this CTA is the state's only reader
      auto input = [&](int i, float (&x)[P]) {          // the input under tap i
        const int src = t - keep + i;                   // its index inside the portion; negative: in front of it
        const float* xp = src >= 0 ? p.in + (s_r0 + src) * (int64_t)p.ldi + col : st + (int64_t)(keep + src) * C;
        const bool none = src < 0 && s_fresh;
        if constexpr (P == 4) {
          const float4 v = none ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(xp);
          x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w;
        } else {
          x[0] = none ? 0.f : *xp;
        }
        if (src >= 0)
#pragma unroll
          for (int e = 0; e < P; ++e) x[e] += b[e];
      };
      auto apply = [&](int i, const float (&x)[P]) {
        const float* wp = cv.w + (int64_t)i * C + c;
        if constexpr (P == 4) {
          const float4 w = __ldg(reinterpret_cast<const float4*>(wp));
          y[0] = fmaf(w.x, x[0], y[0]); y[1] = fmaf(w.y, x[1], y[1]); y[2] = fmaf(w.z, x[2], y[2]); y[3] = fmaf(w.w, x[3], y[3]);
        } else {
          y[0] = fmaf(__ldg(wp), x[0], y[0]);
        }
        if (shift && i > 0) {                           // input i becomes input i - 1 of the next step (read before, by this thread)
          float* dp = st + (int64_t)(i - 1) * C;
          if constexpr (P == 4) *reinterpret_cast<float4*>(dp) = make_float4(x[0], x[1], x[2], x[3]);
          else *dp = x[0];
        }
      };
      if constexpr (TAPS > 0) {
        float x[TAPS][P];
#pragma unroll
        for (int i = 0; i < TAPS; ++i) input(i, x[i]);
#pragma unroll
        for (int i = 0; i < TAPS; ++i) apply(i, x[i]);
      } else {
        for (int i = 0; i < taps; ++i) {
          float x[P];
          input(i, x);
          apply(i, x);
        }
      }
    } else {
#pragma unroll
      for (int e = 0; e < P; ++e) y[e] = p.in[n * p.ldi + col + e] + b[e];
    }
#pragma unroll
    for (int e = 0; e < P; ++e) {
      if (p.act == NVC_PREP_ACT_SILU) y[e] *= sigmoid_f32(y[e]);
      if (P == 1) row[c] = y[e];
      if (c + e < qw) sq += y[e] * y[e];
      else if (c + e < qw + kw) sk += y[e] * y[e];
    }
    if constexpr (P == 4) *reinterpret_cast<float4*>(row + c) = make_float4(y[0], y[1], y[2], y[3]);
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) { part[0][threadIdx.x >> 5] = sq; part[1][threadIdx.x >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) { sq += part[0][w]; sk += part[1][w]; }
  const float rq = p.q_norm ? 1.0f / sqrtf(sq / (float)qw + p.eps) : 1.f, rk = p.k_norm ? 1.0f / sqrtf(sk / (float)kw + p.eps) : 1.f;
  const int half = p.rot_dims >> 1;
  const float2* tab = reinterpret_cast<const float2*>(p.rot_table) + (int64_t)(p.rot_dims ? p.positions[n] : 0) * half;
  for (int c = P * threadIdx.x; c < C; c += step) {
    float y[P];
    if (c >= qw + kw) {
      if (orow < 0) continue;
#pragma unroll
      for (int e = 0; e < P; ++e) y[e] = row[c + e] * p.v_scale;
      TKV* o = reinterpret_cast<TKV*>(p.v_out) + orow * p.ldv + c - qw - kw;
      if constexpr (P == 4) store4(o, make_float4(y[0], y[1], y[2], y[3]));
      else st_f(o, y[0]);
      continue;
    }
    const bool is_q = c < qw;
    if (!is_q && orow < 0) continue;
    const int c0 = is_q ? 0 : qw, cc = c - c0, j0 = cc % p.dim;
    const float r = is_q ? rq : rk, post = is_q ? 1.f : p.k_scale;
    const float* nw = is_q ? p.q_norm : p.k_norm;
    const float* x = row + c0;
    if constexpr (P == 4) {
      if (p.rot_dims == 0 || (p.rot_half && (half & 3) == 0)) {      // four neighbours meet four neighbours
        auto normed = [&](int k) {
          float4 v = *reinterpret_cast<const float4*>(x + k);
          const float4 w = nw ? __ldg(reinterpret_cast<const float4*>(nw + k)) : make_float4(1.f, 1.f, 1.f, 1.f);
          v.x = v.x * r * w.x; v.y = v.y * r * w.y; v.z = v.z * r * w.z; v.w = v.w * r * w.w;
          return v;
        };
        float4 z = normed(cc);
        if (j0 < p.rot_dims) {
          const bool lo = j0 < half;
          const float4* cs = reinterpret_cast<const float4*>(tab + (lo ? j0 : j0 - half));
          const float4 t0 = __ldg(cs), t1 = __ldg(cs + 1), q = normed(lo ? cc + half : cc - half);
          const float sign = lo ? -1.f : 1.f;
          z.x = z.x * t0.x + sign * q.x * t0.y;
          z.y = z.y * t0.z + sign * q.y * t0.w;
          z.z = z.z * t1.x + sign * q.z * t1.y;
          z.w = z.w * t1.z + sign * q.w * t1.w;
        }
        z.x *= post; z.y *= post; z.z *= post; z.w *= post;
        if (is_q) store4(reinterpret_cast<TQ*>(p.q_out) + n * p.ldq + cc, z);
        else store4(reinterpret_cast<TKV*>(p.k_out) + orow * p.ldk + cc, z);
        continue;
      }
    }
#pragma unroll
    for (int e = 0; e < P; ++e) {
      const int j = j0 + e, k = cc + e;                 // number inside its head, number inside the projection
      float z = x[k] * r * (nw ? __ldg(nw + k) : 1.f);
      if (j < p.rot_dims) {
        int i, kp;
        float sign;
        if (p.rot_half) { i = j < half ? j : j - half; kp = j < half ? k + half : k - half; sign = j < half ? -1.f : 1.f; }
        else { i = j >> 1; kp = k - j + (j ^ 1); sign = (j & 1) ? 1.f : -1.f; }
        const float2 cs = __ldg(tab + i);
        z = z * cs.x + sign * (x[kp] * r * (nw ? __ldg(nw + kp) : 1.f)) * cs.y;
      }
      y[e] = z * post;
    }
    if (is_q) {
      TQ* o = reinterpret_cast<TQ*>(p.q_out) + n * p.ldq + cc;
      if constexpr (P == 4) store4(o, make_float4(y[0], y[1], y[2], y[3]));
      else st_f(o, y[0]);
    } else {
      TKV* o = reinterpret_cast<TKV*>(p.k_out) + orow * p.ldk + cc;
      if constexpr (P == 4) store4(o, make_float4(y[0], y[1], y[2], y[3]));
      else st_f(o, y[0]);
    }
  }
}

// one warp per (token, head) of a query projection laid out [heads][dim | rot_dim]: the unrotated part goes to out_a, the rotated
// part (turned by the token's position) to out_b
template <typename T>
__global__ void head_split_rot_kernel(const float* __restrict__ in, int ldi, int heads, int dim, int rot_dim, int rot_dims, int rot_half,
                                      const float* __restrict__ rot_table, const int32_t* __restrict__ positions, T* __restrict__ out_a,
                                      int ld_a, int hs_a, T* __restrict__ out_b, int ld_b, int hs_b, int off_b, int N) {
  pdl_trigger();
  pdl_wait();
  const int64_t u = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (u >= (int64_t)N * heads) return;
  const int n = (int)(u / heads), h = (int)(u % heads);
  const float* x = in + (int64_t)n * ldi + (int64_t)h * (dim + rot_dim);
  T* a = out_a + (int64_t)n * ld_a + (int64_t)h * hs_a;
  for (int j = lane; j < dim; j += 32) st_f(a + j, x[j]);
  const float* xr = x + dim;
  T* b = out_b + (int64_t)n * ld_b + (int64_t)h * hs_b + off_b;
  const int half = rot_dims >> 1;
  const float2* tab = reinterpret_cast<const float2*>(rot_table) + (int64_t)(rot_dims ? positions[n] : 0) * half;
  for (int j = lane; j < rot_dim; j += 32) {
    float y = xr[j];
    if (j < rot_dims) {
      int i, partner;
      float sign;
      if (rot_half) { i = j < half ? j : j - half; partner = j < half ? j + half : j - half; sign = j < half ? -1.f : 1.f; }
      else { i = j >> 1; partner = j ^ 1; sign = (j & 1) ? 1.f : -1.f; }
      const float2 cs = __ldg(tab + i);
      y = y * cs.x + sign * xr[partner] * cs.y;
    }
    st_f(b + j, y);
  }
}

// one CTA per token: the sums of squares of the whole query and the whole key projection in one pass (the key rows leave for the cache
// on the way), then the queries.  VEC: every offset, width and stride is a multiple of 4 and the pointers are 16-byte aligned.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) qk_norm_fold_store_kernel(const float* __restrict__ in, int ldi, int q_off, int qw, int k_off, int kw,
                                                                 const float* __restrict__ wqk, float eps, const int32_t* __restrict__ positions,
                                                                 float temp_coef, int temp_every, T* __restrict__ q_out, int ldq,
                                                                 T* __restrict__ cache, int ldc, float* __restrict__ key_scale,
                                                                 const int32_t* __restrict__ slots) {
  constexpr int P = VEC ? 4 : 1;
  constexpr int KEEP = 8;                              // accesses per thread that stay in registers between the passes
  __shared__ float part[2][8];
  pdl_trigger();
  const int64_t n = blockIdx.x;
  const int slot = slots[n];
  const float temp = 1.0f + temp_coef * logf((float)((positions[n] + 1) / temp_every) + 1.0f);
  pdl_wait();
  const float* q = in + n * ldi + q_off;
  const float* k = in + n * ldi + k_off;
  T* row = cache + (int64_t)slot * ldc;
  float sq = 0.f, sk = 0.f;
  float4 keep[KEEP];
  const int step = P * blockDim.x;
#pragma unroll
  for (int c = 0; c < KEEP; ++c) {
    const int j = P * threadIdx.x + c * step;
    if (j < qw) {
      if constexpr (VEC) {
        const float4 v = *reinterpret_cast<const float4*>(q + j);
        keep[c] = v;
        sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      } else {
        keep[c].x = q[j];
        sq += keep[c].x * keep[c].x;
      }
    }
  }
  for (int j = P * threadIdx.x + KEEP * step; j < qw; j += step) {
    if constexpr (VEC) {
      const float4 v = *reinterpret_cast<const float4*>(q + j);
      sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    } else {
      sq += q[j] * q[j];
    }
  }
  if (slot >= 0) {
    for (int j = P * threadIdx.x; j < kw; j += step) {
      if constexpr (VEC) {
        const float4 v = *reinterpret_cast<const float4*>(k + j);
        store4(row + j, v);
        sk += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      } else {
        st_f(row + j, k[j]);
        sk += k[j] * k[j];
      }
    }
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) { part[0][threadIdx.x >> 5] = sq; part[1][threadIdx.x >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) { sq += part[0][w]; sk += part[1][w]; }
  if (threadIdx.x == 0 && slot >= 0) key_scale[slot] = 1.0f / sqrtf(sk / (float)kw + eps);
  const float r = temp / sqrtf(sq / (float)qw + eps);
  T* o = q_out + n * ldq;
#pragma unroll
  for (int c = 0; c < KEEP; ++c) {
    const int j = P * threadIdx.x + c * step;
    if (j < qw) {
      if constexpr (VEC) {
        const float4 w = *reinterpret_cast<const float4*>(wqk + j);
        store4(o + j, make_float4(keep[c].x * r * w.x, keep[c].y * r * w.y, keep[c].z * r * w.z, keep[c].w * r * w.w));
      } else {
        st_f(o + j, keep[c].x * r * wqk[j]);
      }
    }
  }
  for (int j = P * threadIdx.x + KEEP * step; j < qw; j += step) {
    if constexpr (VEC) {
      const float4 v = *reinterpret_cast<const float4*>(q + j), w = *reinterpret_cast<const float4*>(wqk + j);
      store4(o + j, make_float4(v.x * r * w.x, v.y * r * w.y, v.z * r * w.z, v.w * r * w.w));
    } else {
      st_f(o + j, q[j] * r * wqk[j]);
    }
  }
}

template <typename TQ, typename TKV>
int launch_prep(nvc_ctx* ctx, const nvc_qkv_prep* p, int N, void* stream) {
  PrepArgs a{*p, N};
  const int64_t units = (int64_t)N * (p->q_heads + 2 * p->kv_heads);
  const int wmax = p->dim > p->vdim ? p->dim : p->vdim;
  NVC_CUDA_CHECK(ctx, nvc_launch(ctx, qkv_prep_kernel<TQ, TKV>, dim3((unsigned)((units + 3) / 4)), dim3(128), (size_t)4 * wmax * sizeof(float),
                                 nvc_stream(stream), a));
  ctx->launches++;
  return NVC_OK;
}

template <typename TQ, typename TKV, int P, int TAPS>
int launch_prep_token_as(nvc_ctx* ctx, const PrepArgs& a, const nvc_short_conv& cv, void* stream) {
  const nvc_qkv_prep& p = a.p;
  const int C = p.q_heads * p.dim + p.kv_heads * (p.dim + p.vdim);
  const size_t smem = (size_t)C * sizeof(float);
  static bool attr_set = false;
  if (!attr_set && smem > 48 * 1024) {
    NVC_CUDA_CHECK(ctx, cudaFuncSetAttribute(prep_token_kernel<TQ, TKV, P, TAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr_set = true;
  }
  // few rows: one access per thread, so that a row's loads are all in flight at once
  const int units = (C / P + 31) / 32 * 32;
  const int threads = std::min(std::max(units, 64), a.N <= 2 * ctx->num_sms ? 1024 : 256);
  NVC_CUDA_CHECK(ctx, nvc_launch(ctx, prep_token_kernel<TQ, TKV, P, TAPS>, dim3((unsigned)a.N), dim3(threads), smem, nvc_stream(stream), a, cv));
  ctx->launches++;
  return NVC_OK;
}

template <typename TQ, typename TKV>
int launch_prep_token(nvc_ctx* ctx, const nvc_qkv_prep* p, int N, void* stream) {
  PrepArgs a{*p, N};
  nvc_short_conv cv{};
  if (p->conv) cv = *p->conv;
  const int kw = p->kv_heads * p->dim, vw = p->kv_heads * p->vdim;
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = ((p->dim | kw | vw | p->q_off | p->k_off | p->v_off | p->ldi | p->ldq | p->ldk | p->ldv) & 3) == 0 && al16(p->in) && al16(p->bias) &&
                   al16(cv.w) && al16(cv.state) && al16(p->q_norm) && al16(p->k_norm) && al16(p->rot_table) && al16(p->q_out) && al16(p->k_out) && al16(p->v_out);
  if (!vec) return launch_prep_token_as<TQ, TKV, 1, 0>(ctx, a, cv, stream);
  switch (cv.w ? cv.taps : 0) {
    case 2: return launch_prep_token_as<TQ, TKV, 4, 2>(ctx, a, cv, stream);
    case 3: return launch_prep_token_as<TQ, TKV, 4, 3>(ctx, a, cv, stream);
    case 4: return launch_prep_token_as<TQ, TKV, 4, 4>(ctx, a, cv, stream);
    default: return launch_prep_token_as<TQ, TKV, 4, 0>(ctx, a, cv, stream);
  }
}

}  // namespace

extern "C" int nvc_qkv_prep_run(nvc_ctx* ctx, const nvc_qkv_prep* p, int N, void* stream) {
  NVC_REQUIRE(ctx, ctx && p && p->in && p->q_out && p->k_out && p->v_out, NVC_EINVAL, "null pointer");
  NVC_REQUIRE(ctx, N >= 0 && p->q_heads > 0 && p->kv_heads > 0 && p->dim > 0 && p->vdim > 0 && p->dim <= 2048 && p->vdim <= 2048,
              NVC_EINVAL, "bad sizes");
  NVC_REQUIRE(ctx, p->rot_dims >= 0 && p->rot_dims % 2 == 0 && p->rot_dims <= p->dim && (p->rot_dims == 0 || (p->rot_table && p->positions)),
              NVC_EINVAL, "bad rotary arguments");
  NVC_REQUIRE(ctx, (p->q_norm == nullptr) == (p->k_norm == nullptr) && !(p->unit_norm && p->q_norm), NVC_EINVAL,
              "q and k norms come together, with a weight or without");
  NVC_REQUIRE(ctx, p->blend == NVC_BLEND_NONE || (p->v_first && p->ldvf >= p->kv_heads * p->vdim && (p->blend != NVC_BLEND_MIX || p->lambda)),
              NVC_EINVAL, "value blending needs its buffer and weight");
  NVC_REQUIRE(ctx, p->ldq >= p->q_heads * p->dim && p->ldk >= p->kv_heads * p->dim && p->ldv >= p->kv_heads * p->vdim, NVC_EINVAL,
              "bad strides");
  if (p->conv) {
    const nvc_short_conv& cv = *p->conv;
    NVC_REQUIRE(ctx, cv.w && cv.state && cv.state_slots && p->positions && cv.taps >= 1 && cv.taps <= 16 && cv.B > 0 && (cv.cu_seqlens || N == cv.B),
                NVC_EINVAL, "bad convolution arguments");
    NVC_REQUIRE(ctx, p->k_off == p->q_off + p->q_heads * p->dim && p->v_off == p->k_off + p->kv_heads * p->dim, NVC_EINVAL,
                "a convolution reads neighbouring q, k and v columns");
  }
  if (N == 0) return NVC_OK;
  if (p->conv || p->wide_norm) {
    NVC_REQUIRE(ctx, p->blend == NVC_BLEND_NONE && !p->unit_norm && (p->wide_norm || !p->q_norm), NVC_ENOTIMPL,
                "a convolution goes with whole-projection norms or none, and without blending");
    NVC_REQUIRE(ctx, (size_t)(p->q_heads * p->dim + p->kv_heads * (p->dim + p->vdim)) * sizeof(float) <= 200 * 1024, NVC_ESHAPE,
                "q, k and v of one token above 200 KB");
    if (p->q_dtype == NVC_DT_F32 && p->kv_dtype == NVC_DT_F32) return launch_prep_token<float, float>(ctx, p, N, stream);
    if (p->q_dtype == NVC_DT_BF16 && p->kv_dtype == NVC_DT_BF16) return launch_prep_token<__nv_bfloat16, __nv_bfloat16>(ctx, p, N, stream);
    return NVC_ENOTIMPL;
  }
  {
    auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
    const int qw = p->q_heads * p->dim, kw = p->kv_heads * p->dim, vw = p->kv_heads * p->vdim;
    const bool flat = p->q_dtype == NVC_DT_F32 && p->kv_dtype == NVC_DT_F32 && !p->q_norm && !p->unit_norm && p->rot_dims == 0 &&
                      p->blend == NVC_BLEND_NONE && !p->slot_mapping && p->k_scale == 1.f && p->v_scale == 1.f &&
                      ((qw | kw | vw | p->q_off | p->k_off | p->v_off | p->ldi | p->ldq | p->ldk | p->ldv) & 3) == 0 && al16(p->in) &&
                      al16(p->bias) && al16(p->q_out) && al16(p->k_out) && al16(p->v_out);
    if (flat) {
      PrepArgs a{*p, N};
      NVC_CUDA_CHECK(ctx, nvc_launch(ctx, prep_flat_kernel, dim3((unsigned)N, (unsigned)(((qw + kw + vw) / 4 + 255) / 256)), dim3(256), 0,
                                     nvc_stream(stream), a));
      ctx->launches++;
      return NVC_OK;
    }
  }
  if (p->q_dtype == NVC_DT_F32 && p->kv_dtype == NVC_DT_F32) return launch_prep<float, float>(ctx, p, N, stream);
  if (p->q_dtype == NVC_DT_BF16 && p->kv_dtype == NVC_DT_BF16) return launch_prep<__nv_bfloat16, __nv_bfloat16>(ctx, p, N, stream);
  if (p->q_dtype == NVC_DT_BF16 && p->kv_dtype == NVC_DT_F32) return launch_prep<__nv_bfloat16, float>(ctx, p, N, stream);
  return launch_prep<float, __nv_bfloat16>(ctx, p, N, stream);
}

extern "C" int nvc_head_split_rot(nvc_ctx* ctx, const float* in, int ldi, int heads, int dim, int rot_dim, int rot_dims, int rot_half,
                                  const float* rot_table, const int32_t* positions, void* out_a, int ld_a, int hs_a, void* out_b, int ld_b,
                                  int hs_b, int off_b, int dtype, int N, void* stream) {
  NVC_REQUIRE(ctx, ctx && in && out_a && out_b, NVC_EINVAL, "null pointer");
  NVC_REQUIRE(ctx, N >= 0 && heads > 0 && dim > 0 && rot_dim >= 0 && ldi >= heads * (dim + rot_dim) && hs_a >= dim &&
                       ld_a >= (heads - 1) * hs_a + dim && off_b >= 0 && hs_b >= off_b + rot_dim && ld_b >= (heads - 1) * hs_b + off_b + rot_dim,
              NVC_EINVAL, "bad sizes");
  NVC_REQUIRE(ctx, rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= rot_dim && (rot_dims == 0 || (rot_table && positions)), NVC_EINVAL,
              "bad rotary arguments");
  if (N == 0) return NVC_OK;
  const int64_t units = (int64_t)N * heads;
  NVC_DISPATCH_DT(dtype, T,
                  NVC_CUDA_CHECK(ctx, nvc_launch(ctx, head_split_rot_kernel<T>, dim3((unsigned)((units + 3) / 4)), dim3(128), 0, nvc_stream(stream),
                                                 in, ldi, heads, dim, rot_dim, rot_dims, rot_half, rot_table, positions,
                                                 reinterpret_cast<T*>(out_a), ld_a, hs_a, reinterpret_cast<T*>(out_b), ld_b, hs_b, off_b, N)));
  ctx->launches++;
  return NVC_OK;
}

// (cos, sin) of position * base^(-2 i / dims) for every position below max_pos and i < dims / 2, angles in double precision; with YaRN
// scaling the slow pairs turn `factor` times slower, the fast ones as before and those between the two bounds in part, and cos and sin
// carry one common factor.  Synchronous (called once, when a model is built).
extern "C" int nvc_rotary_table_init_scaled_sync(nvc_ctx* ctx, double base, int dims, nvc_rotary_scaling sc, int max_pos, float* out) {
  NVC_REQUIRE(ctx, ctx && out && dims > 0 && dims % 2 == 0 && max_pos > 0 && base > 0.0, NVC_EINVAL, "bad arguments");
  const bool yarn = sc.factor != 0.0;
  NVC_REQUIRE(ctx, !yarn || (sc.factor > 0.0 && sc.original > 0.0 && sc.fast > 0.0 && sc.slow > 0.0 && base != 1.0), NVC_EINVAL, "bad scaling");
  constexpr double kPi = 3.14159265358979323846;
  auto pair_of = [&](double turns) { return dims * log(sc.original / (2.0 * kPi * turns)) / (2.0 * log(base)); };
  const double lo = yarn ? std::max(floor(pair_of(sc.fast)), 0.0) : 0.0, hi = yarn ? std::min(ceil(pair_of(sc.slow)), (double)(dims - 1)) : 0.0;
  const double mag = yarn ? 0.1 * log(sc.factor) + 1.0 : 1.0;
  const int half = dims / 2;
  std::string buf((size_t)max_pos * half * 2 * sizeof(float), '\0');
  float* h = reinterpret_cast<float*>(&buf[0]);
  for (int i = 0; i < half; ++i) {
    double f = pow(base, -2.0 * (double)i / (double)dims);
    if (yarn) {
      const double ramp = std::min(std::max(((double)i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
      f = f / sc.factor * ramp + f * (1.0 - ramp);
    }
    for (int p = 0; p < max_pos; ++p) {
      const double ang = (double)p * f;
      h[((size_t)p * half + i) * 2] = (float)(cos(ang) * mag);
      h[((size_t)p * half + i) * 2 + 1] = (float)(sin(ang) * mag);
    }
  }
  NVC_CUDA_CHECK(ctx, cudaMemcpy(out, h, buf.size(), cudaMemcpyHostToDevice));
  return NVC_OK;
}

extern "C" int nvc_rotary_table_init_sync(nvc_ctx* ctx, float base, int dims, int max_pos, float* out) {
  return nvc_rotary_table_init_scaled_sync(ctx, (double)base, dims, nvc_rotary_scaling{0.0, 0.0, 0.0, 0.0}, max_pos, out);
}

extern "C" int nvc_qk_norm_fold_store(nvc_ctx* ctx, const float* in, int ldi, int q_off, int qw, int k_off, int kw, const float* wqk, float eps,
                                      const int32_t* positions, float temp_coef, int temp_every, void* q_out, int ldq, void* cache, int ldc,
                                      float* key_scale, const int32_t* slot_mapping, int dtype, int N, void* stream) {
  NVC_REQUIRE(ctx, ctx && in && wqk && positions && q_out && cache && key_scale && slot_mapping, NVC_EINVAL, "null pointer");
  NVC_REQUIRE(ctx, N >= 0 && qw > 0 && kw > 0 && q_off >= 0 && k_off >= 0 && ldi >= q_off + qw && ldi >= k_off + kw && ldq >= qw && ldc >= kw &&
                       temp_every > 0,
              NVC_EINVAL, "bad sizes");
  if (N == 0) return NVC_OK;
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = ((ldi | q_off | qw | k_off | kw | ldq | ldc) & 3) == 0 && al16(in) && al16(wqk) && al16(q_out) && al16(cache);
  const int units = (qw + kw) / (vec ? 4 : 1);
  const int threads = units >= 512 ? 256 : (units >= 192 ? 128 : 64);
  NVC_DISPATCH_DT(dtype, T, {
    auto kv = qk_norm_fold_store_kernel<T, true>;
    auto k1 = qk_norm_fold_store_kernel<T, false>;
    NVC_CUDA_CHECK(ctx, nvc_launch(ctx, vec ? kv : k1, dim3((unsigned)N), dim3((unsigned)threads), 0, nvc_stream(stream), in, ldi, q_off, qw, k_off, kw, wqk,
                                   eps, positions, temp_coef, temp_every, reinterpret_cast<T*>(q_out), ldq, reinterpret_cast<T*>(cache), ldc, key_scale,
                                   slot_mapping));
  });
  ctx->launches++;
  return NVC_OK;
}
