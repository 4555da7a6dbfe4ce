// The gated delta rule: a linear-attention mixer whose per-head state S [dim, vdim] is decayed, corrected towards the new value
// and read in every token,
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q,
// with q, k, v taken through a short causal convolution over time per channel.  Three kernels:
//   delta_prep_kernel   one warp per (token, unit), the sequence from the block index: convolution + silu of a q / k / v head (the taps - 1 inputs in front of a
//                       portion come from the sequence's convolution state), unit length for q and k, q scale; one more unit per token
//                       for the per-head decay g = exp(-exp(A_log) softplus(a + dt_bias)) and beta = sigmoid(b)
//   delta_scan_kernel   one CTA per (sequence, head, slice of 32 value columns); thread (column v, row group r) keeps rows
//                       [r DPT, (r + 1) DPT) of column v of the state in registers and walks the sequence's new tokens.  One pass over
//                       the state per token: with a = S^T k, c = S^T q of the state BEFORE the token and kq = k . q,
//                           u = beta (v - g a),   o = g c + kq u,   S <- g S + k u^T
//                       (the same sums as the four steps above, regrouped so that a token needs one reduction over row groups).
//                       The CTAs of a sequence also advance its convolution state, a share of the channels each.
//   delta_chunk_kernel  the same recurrence 32 tokens at a time for prompt portions (see there).
// With a decay per head and key CHANNEL (g a vector, S <- diag(g) S) the token kernel scales every row of S first and then follows the
// four steps, and the chunk kernel works with the running sums L_t of each channel: the token-by-token products take
// exp(L_t - L_j) inside their sums, the keys and queries that meet the state carry exp(L_t), those that enter it exp(L_n - L_j).
// Both states live in fp32 in pools of state slots; a sequence whose first new token sits at position 0 starts from zeros.
// Everything here is plain fp32 FMA code.
#include <type_traits>

#include "scan_common.cuh"

namespace {

struct DeltaArgs {
  nvc_delta_prep p;
  int N;
  int vec;                       // sizes, strides and pointers allow 16-byte accesses
  float* o;
  int ldo;
  float* state;
};

__device__ __forceinline__ float softplus_f32(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// grid (token tiles of the longest portion, units, sequences): the sequence comes from the block index, so a warp's first loads are
// its sequence's bounds and nothing has to be searched; CTAs behind a sequence's last token leave at once
// TAPS: the convolution's taps when they are 2 .. 4 (all inputs of a channel are in flight at once), 0: any number of them
template <int TAPS>
__global__ void __launch_bounds__(128, 8) delta_prep_kernel(const DeltaArgs a) {
  pdl_trigger();
  pdl_wait();
  const nvc_delta_prep& p = a.p;
  const int wid = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int units = 2 * p.kv_heads + p.heads + 1;
  const int b = blockIdx.z, uu = blockIdx.y;
  const int r0 = p.cu_seqlens ? p.cu_seqlens[b] : b;
  const int r1 = p.cu_seqlens ? p.cu_seqlens[b + 1] : b + 1;
  const int n = r0 + blockIdx.x * (blockDim.x >> 5) + wid;
  if (n >= r1) return;
  const float* in = p.in + (int64_t)n * p.ldi;
  if (uu >= units) {
    // ---- log decays of one head's key channels
    const int h = uu - units;
    const float* x = p.channel_a + (int64_t)n * p.ldca + h * p.dim;
    const float* bias = p.dt_bias + h * p.dim;
    float* g = p.channel_g + ((int64_t)n * p.heads + h) * p.dim;
    const float na = -expf(__ldg(p.A_log + h));
    if (a.vec && (p.ldca & 3) == 0) {
      for (int j = 4 * lane; j < p.dim; j += 128) {
        const float4 v = *reinterpret_cast<const float4*>(x + j), u = __ldg(reinterpret_cast<const float4*>(bias + j));
        *reinterpret_cast<float4*>(g + j) =
            make_float4(na * softplus_f32(v.x + u.x), na * softplus_f32(v.y + u.y), na * softplus_f32(v.z + u.z), na * softplus_f32(v.w + u.w));
      }
    } else {
      for (int j = lane; j < p.dim; j += 32) g[j] = na * softplus_f32(x[j] + __ldg(bias + j));
    }
    return;
  }
  if (uu == units - 1) {
    // ---- decay and beta of every head
    for (int h = lane; h < p.heads; h += 32) {
      if (p.channel_a) {
        p.gb_out[(int64_t)n * 2 * p.heads + 2 * h + 1] = sigmoid_f32(in[p.b_off + h]);
        continue;
      }
      const float dt = softplus_f32(in[p.a_off + h] + __ldg(p.dt_bias + h));
      p.gb_out[(int64_t)n * 2 * p.heads + 2 * h] = -expf(__ldg(p.A_log + h)) * dt;       // log of the decay
      p.gb_out[(int64_t)n * 2 * p.heads + 2 * h + 1] = sigmoid_f32(in[p.b_off + h]);
    }
    return;
  }
  const int t = n - r0;                                 // index inside the portion
  const bool fresh = p.positions[r0] == 0;
  const int C = 2 * p.kv_heads * p.dim + p.heads * p.vdim;
  const float* cs = p.conv_state + (int64_t)p.state_slots[b] * (p.taps - 1) * C;
  // which head: q heads, then k heads, then v heads
  int kind, h;
  if (uu < p.kv_heads) { kind = 0; h = uu; }
  else if (uu < 2 * p.kv_heads) { kind = 1; h = uu - p.kv_heads; }
  else { kind = 2; h = uu - 2 * p.kv_heads; }
  const int width = kind == 2 ? p.vdim : p.dim;
  const int col = (kind == 0 ? p.q_off : (kind == 1 ? p.k_off : p.v_off)) + h * width;            // column of the projection row
  const int ch = (kind == 0 ? 0 : (kind == 1 ? p.kv_heads * p.dim : 2 * p.kv_heads * p.dim)) + h * width;   // channel
  float* out = kind == 0 ? p.q_out + (int64_t)n * p.ldq : (kind == 1 ? p.k_out + (int64_t)n * p.ldk : p.v_out + (int64_t)n * p.ldv);
  out += h * width;
  if (a.vec && width <= 512) {
    // four channels per lane, 16-byte accesses, the head stays in registers between the convolution and the unit length
    float4 y[4];
    float ss4 = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int j = 4 * lane + 128 * k;
      y[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (j < width) {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        const int taps = TAPS > 0 ? TAPS : p.taps;
        auto input = [&](int i) {          // the input under tap i
          const int src = t - (taps - 1) + i;
          const float* xp = src >= 0 ? in + (int64_t)(src - t) * p.ldi + col + j : cs + (int64_t)(taps - 1 + src) * C + ch + j;
          return (src < 0 && fresh) ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(xp);
        };
        auto apply = [&](int i, const float4& x) {
          const float4 w = __ldg(reinterpret_cast<const float4*>(p.conv_w + (int64_t)i * C + ch + j));      // tap-major: lanes read side by side
          acc.x = fmaf(w.x, x.x, acc.x);
          acc.y = fmaf(w.y, x.y, acc.y);
          acc.z = fmaf(w.z, x.z, acc.z);
          acc.w = fmaf(w.w, x.w, acc.w);
        };
        if constexpr (TAPS > 0) {
          float4 x[TAPS];
#pragma unroll
          for (int i = 0; i < TAPS; ++i) x[i] = input(i);
#pragma unroll
          for (int i = 0; i < TAPS; ++i) apply(i, x[i]);
        } else {
          for (int i = 0; i < taps; ++i) apply(i, input(i));
        }
        y[k] = make_float4(acc.x * sigmoid_f32(acc.x), acc.y * sigmoid_f32(acc.y), acc.z * sigmoid_f32(acc.z), acc.w * sigmoid_f32(acc.w));
        ss4 += y[k].x * y[k].x + y[k].y * y[k].y + y[k].z * y[k].z + y[k].w * y[k].w;
      }
    }
    float r = 1.f;
    if (kind != 2) r = (kind == 0 ? p.q_scale : 1.f) / sqrtf(warp_sum(ss4) + p.unit_eps);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int j = 4 * lane + 128 * k;
      if (j < width) *reinterpret_cast<float4*>(out + j) = make_float4(y[k].x * r, y[k].y * r, y[k].z * r, y[k].w * r);
    }
    return;
  }
  float ss = 0.f;
  for (int j = lane; j < width; j += 32) {
    float acc = 0.f;
    for (int i = 0; i < p.taps; ++i) {
      const int src = t - (p.taps - 1) + i;             // portion index of the input under tap i
      float x;
      if (src >= 0) x = in[(int64_t)(src - t) * p.ldi + col + j];
      else x = fresh ? 0.f : cs[(int64_t)(p.taps - 1 + src) * C + ch + j];
      acc = fmaf(__ldg(p.conv_w + (int64_t)i * C + ch + j), x, acc);
    }
    const float y = acc * sigmoid_f32(acc);
    out[j] = y;
    ss += y * y;
  }
  if (kind == 2) return;
  ss = warp_sum(ss);
  const float r = (kind == 0 ? p.q_scale : 1.f) / sqrtf(ss + p.unit_eps);
  __syncwarp();
  for (int j = lane; j < width; j += 32) out[j] *= r;
}


// The convolution state of a sequence after a portion: the last taps - 1 inputs of (what it held, this portion).  Slot i reads slot
// i + len or the portion, never a slot below itself, so one thread per channel shifts in place.  The channels are spread over the
// CTAs (head, value slice) of the sequence; nothing else in a scan kernel reads this state.
__device__ __forceinline__ void advance_conv_state(const nvc_delta_prep& p, int r0, int r1, bool fresh, int slot) {
  const int C = 2 * p.kv_heads * p.dim + p.heads * p.vdim, len = r1 - r0, keep = p.taps - 1;
  if (keep == 0) return;
  float* cs = p.conv_state + (int64_t)slot * keep * C;
  const int part = blockIdx.y * gridDim.z + blockIdx.z, parts = gridDim.y * gridDim.z;
  const int qk = p.kv_heads * p.dim;
  for (int c = part * blockDim.x + threadIdx.x; c < C; c += parts * blockDim.x) {
    const int col = c < qk ? p.q_off + c : (c < 2 * qk ? p.k_off + c - qk : p.v_off + c - 2 * qk);
    for (int i = 0; i < keep; ++i) {
      const int src = len - keep + i;                 // portion index
      float x;
      if (src >= 0) x = p.in[(int64_t)(r0 + src) * p.ldi + col];
      else x = fresh ? 0.f : cs[(int64_t)(keep + src) * C + c];
      cs[(int64_t)i * C + c] = x;
    }
  }
}

// CH: a decay per key channel
template <int DPT, bool CH>
__global__ void delta_scan_kernel(const DeltaArgs a) {
  extern __shared__ float sm[];
  pdl_trigger();
  const nvc_delta_prep& p = a.p;
  const int b = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * 32;
  const int lane = threadIdx.x & 31, rg = threadIdx.x >> 5, groups = blockDim.x >> 5;
  const int v = v0 + lane;
  const bool vok = v < p.vdim;
  const int hk = h / (p.heads / p.kv_heads);
  float* q_s = sm;                    // [2][dim]
  float* k_s = sm + 2 * p.dim;        // [2][dim]
  float* g_s = sm + 4 * p.dim;        // [2][dim] (CH): decays
  float* red = sm + (CH ? 6 : 4) * p.dim;        // [3][groups][32]
  pdl_wait();
  const int r0 = p.cu_seqlens ? p.cu_seqlens[b] : b;
  const int r1 = p.cu_seqlens ? p.cu_seqlens[b + 1] : b + 1;
  const bool fresh = p.positions[r0] == 0;
  const int slot = p.state_slots[b];
  advance_conv_state(p, r0, r1, fresh, slot);
  const int d0 = rg * DPT;
  float S[DPT];
  float* sp = a.state + (((int64_t)slot * p.heads + h) * p.dim) * p.vdim;
#pragma unroll
  for (int i = 0; i < DPT; ++i) S[i] = (!fresh && vok && d0 + i < p.dim) ? sp[(int64_t)(d0 + i) * p.vdim + v] : 0.f;
  for (int d = threadIdx.x; d < p.dim; d += blockDim.x) {
    q_s[d] = p.q_out[(int64_t)r0 * p.ldq + hk * p.dim + d];
    k_s[d] = p.k_out[(int64_t)r0 * p.ldk + hk * p.dim + d];
    if (CH) g_s[d] = expf(p.channel_g[((int64_t)r0 * p.heads + h) * p.dim + d]);
  }
  float vt = vok ? p.v_out[(int64_t)r0 * p.ldv + h * p.vdim + v] : 0.f;
  float gt = CH ? 1.f : expf(p.gb_out[(int64_t)r0 * 2 * p.heads + 2 * h]), bt = p.gb_out[(int64_t)r0 * 2 * p.heads + 2 * h + 1];
  __syncthreads();
  for (int t = r0; t < r1; ++t) {
    const int cur = (t - r0) & 1;
    const float* qc = q_s + cur * p.dim;
    const float* kc = k_s + cur * p.dim;
    float vn = 0.f, gn = 0.f, bn = 0.f;
    if (t + 1 < r1) {       // fetch the next token into the other buffer
      for (int d = threadIdx.x; d < p.dim; d += blockDim.x) {
        q_s[(cur ^ 1) * p.dim + d] = p.q_out[(int64_t)(t + 1) * p.ldq + hk * p.dim + d];
        k_s[(cur ^ 1) * p.dim + d] = p.k_out[(int64_t)(t + 1) * p.ldk + hk * p.dim + d];
        if (CH) g_s[(cur ^ 1) * p.dim + d] = expf(p.channel_g[((int64_t)(t + 1) * p.heads + h) * p.dim + d]);
      }
      vn = vok ? p.v_out[(int64_t)(t + 1) * p.ldv + h * p.vdim + v] : 0.f;
      if (!CH) gn = expf(p.gb_out[(int64_t)(t + 1) * 2 * p.heads + 2 * h]);
      bn = p.gb_out[(int64_t)(t + 1) * 2 * p.heads + 2 * h + 1];
    }
    float sk = 0.f, sq = 0.f, kq = 0.f;
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
      if (d0 + i < p.dim) {
        const float kv = kc[d0 + i], qv = qc[d0 + i];
        if (CH) S[i] *= g_s[cur * p.dim + d0 + i];
        sk = fmaf(S[i], kv, sk);
        sq = fmaf(S[i], qv, sq);
        kq = fmaf(kv, qv, kq);
      }
    }
    if (groups > 1) {
      red[(0 * groups + rg) * 32 + lane] = sk;
      red[(1 * groups + rg) * 32 + lane] = sq;
      red[(2 * groups + rg) * 32 + lane] = kq;
      __syncthreads();
      sk = sq = kq = 0.f;
      for (int g = 0; g < groups; ++g) {
        sk += red[(0 * groups + g) * 32 + lane];
        sq += red[(1 * groups + g) * 32 + lane];
        kq += red[(2 * groups + g) * 32 + lane];
      }
    }
    if (CH) gt = 1.f;                 // the decay is in the rows already
    const float u = bt * (vt - gt * sk);
    if (vok && rg == 0) a.o[(int64_t)t * a.ldo + h * p.vdim + v] = fmaf(kq, u, gt * sq);
#pragma unroll
    for (int i = 0; i < DPT; ++i)
      if (d0 + i < p.dim) S[i] = fmaf(gt, S[i], kc[d0 + i] * u);
    vt = vn; gt = gn; bt = bn;
    __syncthreads();
  }
  if (vok)
#pragma unroll
    for (int i = 0; i < DPT; ++i)
      if (d0 + i < p.dim) sp[(int64_t)(d0 + i) * p.vdim + v] = S[i];
}


// ---- prompt portions: 16 tokens at a time.  Within a chunk that starts from the state S0, with L_t the running sum of log g up to
// token t (so exp(L_t - L_j) is the decay between tokens j and t; a number, or one per key channel),
//   u_t = beta_t (v_t - S0^T (exp(L_t) k_t) - sum_{j<t} (k_t . exp(L_t - L_j) k_j) u_j)      a unit lower triangular system
//   o_t = S0^T (exp(L_t) q_t) + sum_{j<=t} (q_t . exp(L_t - L_j) k_j) u_j
//   S   = exp(L_n) S0 + sum_j (exp(L_n - L_j) k_j) u_j^T
// which are the four steps of the recurrence written out over the chunk; only differences L_t - L_j <= 0 are exponentiated, so a
// decay that underflows over a chunk stays a plain zero.  (A product of two one-sided factors would not do for the token-by-token
// terms of a channel: exp(-L_j) overflows.  That, and the exponentials it costs, is why a chunk is no longer than 16 tokens.)
// One CTA per (sequence, head, COLS = 32 C NW / 4 value columns); the state slice stays in shared memory.  Stages of a chunk:
//   copy      k, q (and log decays) of the chunk, asynchronously; running sums by one thread per channel
//   products  token against token, lanes along the channels, a warp takes whole rows t; A is kept transposed (AT)
//   scale     (channels) the rows that meet the state get exp(L_t), those that enter it exp(L_n - L_t)
//   state     a warp takes 8 of the 32 rows [k | q] against 32 C columns of the state: 8 C sums per thread
//   solve     forward substitution, column by column of A (every step updates all later right sides: no long dependent sums)
//   outputs by the warps that hold the query rows' sums, then the state update, 8 rows x C columns at a time
// Tokens behind a portion's end are padded with g = 1, beta = 0, k = q = v = 0, which leaves state and outputs alone.
constexpr int kDT = 16;                  // tokens per chunk
constexpr int kDA = kDT + 4;             // row stride of the token-by-token matrices (16-byte rows)

__host__ __device__ inline size_t delta_chunk_smem_floats(int dim, int cols, bool channels) {
  const int dz = scan_row(dim);
  return (size_t)(channels ? 3 : 2) * kDT * (dz + 4) + 2 * kDT * kDA + (size_t)kDT * cols + (size_t)dz * cols + dz + 2 * kDT;
}

template <int C, int NW, bool CH>
__global__ void __launch_bounds__(NW * 32, NW == 8 ? 2 : 3) delta_chunk_kernel(const DeltaArgs a) {
  constexpr int COLS = 32 * C * (NW / 4), THREADS = NW * 32;
  constexpr float kLog2e = 1.4426950408889634f;
  extern __shared__ __align__(16) float sm[];
  pdl_trigger();
  const nvc_delta_prep& p = a.p;
  const int b = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * COLS;
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, rg = w & 3;
  const int hk = h / (p.heads / p.kv_heads);
  const int dim = p.dim, dz = scan_row(dim), ds = dz + 4;
  float* Ks = sm;                          // [16][ds]
  float* Qs = Ks + kDT * ds;               // [16][ds]
  float* Gs = Qs + kDT * ds;               // [16][ds] (CH) running sums of the log2 decays, later exp(L_t) k_t
  float* AT = Gs + (CH ? kDT * ds : 0);    // [16][20] AT[j][t] = beta_t (k_t . exp(L_t - L_j) k_j), t > j, else 0
  float* Pm = AT + kDT * kDA;              // [16][20] Pm[t][j] = q_t . exp(L_t - L_j) k_j, j <= t, else 0
  float* Us = Pm + kDT * kDA;              // [16][COLS] right sides, then u_t
  float* Ss = Us + kDT * COLS;             // [dz][COLS] the state's columns
  float* En = Ss + (size_t)dz * COLS;      // [dz] (CH) log2 decays over the whole chunk
  float* Ls = En + dz;                     // [16] running sums of the head's log2 decays (zeros: CH)
  float* Bs = Ls + kDT;                    // [16]
  pdl_wait();
  const int r0 = p.cu_seqlens ? p.cu_seqlens[b] : b;
  const int r1 = p.cu_seqlens ? p.cu_seqlens[b + 1] : b + 1;
  const bool fresh = p.positions[r0] == 0;
  const int slot = p.state_slots[b];
  advance_conv_state(p, r0, r1, fresh, slot);
  float* sp = a.state + (((int64_t)slot * p.heads + h) * dim) * p.vdim;
  for (int i = threadIdx.x; i < dz * COLS; i += THREADS) {
    const int d = i / COLS, c = i % COLS;
    Ss[i] = (!fresh && d < dim && v0 + c < p.vdim) ? sp[(int64_t)d * p.vdim + v0 + c] : 0.f;
  }
  for (int i = threadIdx.x; i < 2 * kDT * kDA; i += THREADS) AT[i] = 0.f;      // what the products never write stays zero
  const int cl = (w >> 2) * 32 * C + lane * C;             // this lane's first column of the slice
  for (int c0 = r0; c0 < r1; c0 += kDT) {
    const int n = min(kDT, r1 - c0);
    // ---- copy
    const float* kg = p.k_out + (int64_t)c0 * p.ldk + hk * dim;
    const float* qg = p.q_out + (int64_t)c0 * p.ldq + hk * dim;
    const float* gg = CH ? p.channel_g + ((int64_t)c0 * p.heads + h) * dim : nullptr;
    const int ldg = p.heads * dim;
    for (int t = w; t < kDT; t += NW) {
      copy_row(Ks + t * ds, kg + (int64_t)t * p.ldk, dim, dz, t < n, a.vec, lane);
      copy_row(Qs + t * ds, qg + (int64_t)t * p.ldq, dim, dz, t < n, a.vec, lane);
      if (CH) copy_row(Gs + t * ds, gg + (int64_t)t * ldg, dim, dz, t < n, a.vec, lane);
    }
    // what this warp needs of v: the tokens of its key rows (rg 0 and 1)
    float vt[8][C];
    if (rg < 2) {
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        const int t = 8 * rg + r;
        const float* vp = p.v_out + (int64_t)(c0 + t) * p.ldv + h * p.vdim + v0 + cl;
#pragma unroll
        for (int e = 0; e < C; ++e) vt[r][e] = (t < n && v0 + cl + e < p.vdim) ? vp[e] : 0.f;
      }
    }
    if (w == 0 && lane < kDT) {
      const float* gb = p.gb_out + ((int64_t)(c0 + lane) * p.heads + h) * 2;
      float lg = (!CH && lane < n) ? gb[0] * kLog2e : 0.f;
#pragma unroll
      for (int o = 1; o < kDT; o <<= 1) {
        const float up = __shfl_up_sync(0xffffu, lg, o);
        if (lane >= o) lg += up;
      }
      Ls[lane] = lg;
      Bs[lane] = lane < n ? gb[1] : 0.f;
    }
    copy_async_wait();
    __syncthreads();
    if constexpr (CH) {
      for (int c = threadIdx.x; c < dz; c += THREADS) {
        float x[kDT], l = 0.f;
#pragma unroll
        for (int t = 0; t < kDT; ++t) x[t] = Gs[t * ds + c];
#pragma unroll
        for (int t = 0; t < kDT; ++t) { l = fmaf(x[t], kLog2e, l); Gs[t * ds + c] = l; }
        En[c] = l;
      }
      __syncthreads();
    }
    // ---- products: a row t against four earlier tokens at a time, groups of GL lanes along the channels.  The eight sums of a group: k and
    // q against four j.
    {
      const int GL = dz > 64 ? 32 : (dz > 32 ? 16 : 8), gl = lane & (GL - 1), sub = lane / GL, subs = 32 / GL;
#pragma unroll 1
      for (int i = 0; i < kDT / NW; ++i) {                  // rows in pairs that add up to equal work
        const int t = (i & 1) ? (i + 1) * NW - 1 - w : i * NW + w;
        float4 kt[2], qt[2], gt[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int c = 4 * gl + 4 * GL * e;
          kt[e] = qt[e] = gt[e] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (c < dz) {
            kt[e] = *reinterpret_cast<const float4*>(Ks + t * ds + c);
            qt[e] = *reinterpret_cast<const float4*>(Qs + t * ds + c);
            if (CH) gt[e] = *reinterpret_cast<const float4*>(Gs + t * ds + c);
          }
        }
        const float bt = Bs[t], lt = Ls[t];
#pragma unroll 1
        for (int j0 = 0; j0 <= t; j0 += 4 * subs) {
          const int jb = min(j0 + 4 * sub, kDT - 4);        // groups behind the last row repeat it
          float v[8];
#pragma unroll
          for (int y = 0; y < 8; ++y) v[y] = 0.f;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int c = 4 * gl + 4 * GL * e;
            if (c < dz) {
#pragma unroll
              for (int y = 0; y < 4; ++y) {
                float4 x = *reinterpret_cast<const float4*>(Ks + (jb + y) * ds + c);
                if (CH) {                                   // j > t: anything may come out, nothing is kept
                  const float4 g = *reinterpret_cast<const float4*>(Gs + (jb + y) * ds + c);
                  x.x *= ex2(gt[e].x - g.x); x.y *= ex2(gt[e].y - g.y); x.z *= ex2(gt[e].z - g.z); x.w *= ex2(gt[e].w - g.w);
                }
                v[y] = fma4(kt[e], x, v[y]);
                v[4 + y] = fma4(qt[e], x, v[4 + y]);
              }
            }
          }
          int which;
          bool writer;
          const float sum = group_sum8(v, GL, gl, &which, &writer);
          const int j = jb + (which & 3);
          if (writer && j <= t) {
            const float x = CH ? sum : ex2(lt - Ls[j]) * sum;
            if (which >= 4) Pm[t * kDA + j] = x;
            else if (j < t) AT[j * kDA + t] = bt * x;
          }
        }
      }
    }
    if constexpr (CH) {
      __syncthreads();                                      // the products have read the plain rows
      for (int t = w; t < kDT; t += NW)
        for (int c = 4 * lane; c < dz; c += 128) {
          float4 k = *reinterpret_cast<float4*>(Ks + t * ds + c), q = *reinterpret_cast<float4*>(Qs + t * ds + c);
          const float4 l = *reinterpret_cast<float4*>(Gs + t * ds + c), ln = *reinterpret_cast<float4*>(En + c);
          const float4 f = make_float4(ex2(l.x), ex2(l.y), ex2(l.z), ex2(l.w));
          *reinterpret_cast<float4*>(Qs + t * ds + c) = make_float4(q.x * f.x, q.y * f.y, q.z * f.z, q.w * f.w);
          *reinterpret_cast<float4*>(Gs + t * ds + c) = make_float4(k.x * f.x, k.y * f.y, k.z * f.z, k.w * f.w);
          *reinterpret_cast<float4*>(Ks + t * ds + c) =
              make_float4(k.x * ex2(ln.x - l.x), k.y * ex2(ln.y - l.y), k.z * ex2(ln.z - l.z), k.w * ex2(ln.w - l.w));
        }
    }
    __syncthreads();
    // ---- state: rows 0 .. 15 are the keys', 16 .. 31 the queries'
    float acc[8][C];
#pragma unroll
    for (int r = 0; r < 8; ++r)
#pragma unroll
      for (int e = 0; e < C; ++e) acc[r][e] = 0.f;
    {
      const float* X = (rg < 2 ? (CH ? Gs : Ks) : Qs) + (rg & 1) * 8 * ds;
#pragma unroll 2
      for (int d = 0; d < dz; d += 4) {
        float s[4][C];
#pragma unroll
        for (int i = 0; i < 4; ++i) ld_cols<C>(s[i], Ss + (d + i) * COLS + cl);
#pragma unroll
        for (int r = 0; r < 8; ++r) {
          const float4 x = *reinterpret_cast<const float4*>(X + r * ds + d);
#pragma unroll
          for (int e = 0; e < C; ++e) {
            acc[r][e] = fmaf(x.x, s[0][e], acc[r][e]);
            acc[r][e] = fmaf(x.y, s[1][e], acc[r][e]);
            acc[r][e] = fmaf(x.z, s[2][e], acc[r][e]);
            acc[r][e] = fmaf(x.w, s[3][e], acc[r][e]);
          }
        }
      }
    }
    if (rg < 2) {
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        const int t = 8 * rg + r;
        const float bt = Bs[t], f = CH ? 1.f : ex2(Ls[t]);
        float x[C];
#pragma unroll
        for (int e = 0; e < C; ++e) x[e] = bt * (vt[r][e] - f * acc[r][e]);
        st_cols<C>(Us + t * COLS + cl, x);
      }
    }
    __syncthreads();
    // ---- solve: one warp per group of columns
    if (rg == 0) {
      float x[kDT][C];
#pragma unroll
      for (int t = 0; t < kDT; ++t) ld_cols<C>(x[t], Us + t * COLS + cl);
#pragma unroll
      for (int j = 0; j + 1 < kDT; ++j) {
#pragma unroll
        for (int t4 = (j + 1) / 4 * 4; t4 < kDT; t4 += 4) {
          const float4 m = *reinterpret_cast<const float4*>(AT + j * kDA + t4);
#pragma unroll
          for (int e = 0; e < C; ++e) {
            if (t4 > j) x[t4][e] = fmaf(-m.x, x[j][e], x[t4][e]);
            if (t4 + 1 > j) x[t4 + 1][e] = fmaf(-m.y, x[j][e], x[t4 + 1][e]);
            if (t4 + 2 > j) x[t4 + 2][e] = fmaf(-m.z, x[j][e], x[t4 + 2][e]);
            if (t4 + 3 > j) x[t4 + 3][e] = fmaf(-m.w, x[j][e], x[t4 + 3][e]);
          }
        }
      }
#pragma unroll
      for (int t = 1; t < kDT; ++t) st_cols<C>(Us + t * COLS + cl, x[t]);
    }
    __syncthreads();
    // ---- outputs
    float u[kDT][C];
#pragma unroll
    for (int j = 0; j < kDT; ++j) ld_cols<C>(u[j], Us + j * COLS + cl);
    if (rg >= 2) {
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        const int t = 8 * (rg - 2) + r;
        float o[C];
        const float f = CH ? 1.f : ex2(Ls[t]);
#pragma unroll
        for (int e = 0; e < C; ++e) o[e] = f * acc[r][e];
#pragma unroll
        for (int j4 = 0; j4 < kDT; j4 += 4) {               // entries behind the diagonal are zero
          const float4 m = *reinterpret_cast<const float4*>(Pm + t * kDA + j4);
#pragma unroll
          for (int e = 0; e < C; ++e) {
            o[e] = fmaf(m.x, u[j4][e], o[e]);
            o[e] = fmaf(m.y, u[j4 + 1][e], o[e]);
            o[e] = fmaf(m.z, u[j4 + 2][e], o[e]);
            o[e] = fmaf(m.w, u[j4 + 3][e], o[e]);
          }
        }
        float* op = a.o + (int64_t)(c0 + t) * a.ldo + h * p.vdim + v0 + cl;
#pragma unroll
        for (int e = 0; e < C; ++e)
          if (t < n && v0 + cl + e < p.vdim) op[e] = o[e];
      }
    }
    // ---- the state behind the chunk
    if (!CH) {
      const float ln = Ls[kDT - 1];
#pragma unroll
      for (int j = 0; j < kDT; ++j) {
        const float f = ex2(ln - Ls[j]);
#pragma unroll
        for (int e = 0; e < C; ++e) u[j][e] *= f;
      }
    }
    for (int d = 4 * rg; d < dz; d += 16) {
      float s[4][C];
      const float4 g = CH ? *reinterpret_cast<const float4*>(En + d) : make_float4(Ls[kDT - 1], Ls[kDT - 1], Ls[kDT - 1], Ls[kDT - 1]);
      const float f[4] = {ex2(g.x), ex2(g.y), ex2(g.z), ex2(g.w)};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        ld_cols<C>(s[i], Ss + (d + i) * COLS + cl);
#pragma unroll
        for (int e = 0; e < C; ++e) s[i][e] *= f[i];
      }
#pragma unroll
      for (int j = 0; j < kDT; ++j) {
        const float4 k = *reinterpret_cast<const float4*>(Ks + j * ds + d);
#pragma unroll
        for (int e = 0; e < C; ++e) {
          s[0][e] = fmaf(k.x, u[j][e], s[0][e]);
          s[1][e] = fmaf(k.y, u[j][e], s[1][e]);
          s[2][e] = fmaf(k.z, u[j][e], s[2][e]);
          s[3][e] = fmaf(k.w, u[j][e], s[3][e]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) st_cols<C>(Ss + (d + i) * COLS + cl, s[i]);
    }
    __syncthreads();
  }
  for (int i = threadIdx.x; i < dim * COLS; i += THREADS) {
    const int d = i / COLS, c = i % COLS;
    if (v0 + c < p.vdim) sp[(int64_t)d * p.vdim + v0 + c] = Ss[i];
  }
}

template <int C, int NW, bool CH>
cudaError_t launch_delta_chunk(nvc_ctx* ctx, const DeltaArgs& a, cudaStream_t st) {
  constexpr int COLS = 32 * C * (NW / 4);
  const size_t smem = delta_chunk_smem_floats(a.p.dim, COLS, CH) * sizeof(float);
  static bool attr_set = false;
  if (!attr_set && smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(delta_chunk_kernel<C, NW, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) return e;
    attr_set = true;
  }
  return nvc_launch(ctx, delta_chunk_kernel<C, NW, CH>, dim3(a.p.B, a.p.heads, (a.p.vdim + COLS - 1) / COLS), dim3(NW * 32), smem, st, a);
}

// The wider the slice, the less often the token-by-token products of a head are repeated; as long as the slices fill the GPU
template <bool CH>
cudaError_t launch_delta_chunk_sized(nvc_ctx* ctx, const DeltaArgs& a, cudaStream_t st) {
  const int units = a.p.B * a.p.heads, sms = ctx->num_sms;
  if (a.p.vdim > 64 && 4 * units * ((a.p.vdim + 127) / 128) >= 3 * sms) return launch_delta_chunk<2, 8, CH>(ctx, a, st);
  return launch_delta_chunk<1, 8, CH>(ctx, a, st);
}

int check_prep(nvc_ctx* ctx, const nvc_delta_prep* p) {
  NVC_REQUIRE(ctx, ctx && p && p->in && p->conv_w && p->conv_state && p->state_slots && p->positions && p->A_log && p->dt_bias && p->q_out &&
                       p->k_out && p->v_out && p->gb_out, NVC_EINVAL, "null pointer");
  NVC_REQUIRE(ctx, p->heads > 0 && p->kv_heads > 0 && p->heads % p->kv_heads == 0 && p->dim > 0 && p->vdim > 0 && p->taps >= 1 && p->B > 0 &&
                       p->dim <= 1024 && p->heads <= 65535, NVC_EINVAL, "bad sizes");
  NVC_REQUIRE(ctx, p->ldq >= p->kv_heads * p->dim && p->ldk >= p->kv_heads * p->dim && p->ldv >= p->heads * p->vdim, NVC_EINVAL, "bad strides");
  NVC_REQUIRE(ctx, !p->channel_a || (p->channel_g && p->ldca >= p->heads * p->dim), NVC_EINVAL, "decays per channel need their output rows");
  return NVC_OK;
}

}  // namespace

extern "C" int nvc_delta_prep_run(nvc_ctx* ctx, const nvc_delta_prep* p, int N, int max_qlen, void* stream) {
  int rc = check_prep(ctx, p);
  if (rc) return rc;
  NVC_REQUIRE(ctx, p->cu_seqlens || N == p->B, NVC_EINVAL, "rows without cu_seqlens: one per sequence");
  if (N == 0) return NVC_OK;
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const int vec = p->dim % 4 == 0 && p->vdim % 4 == 0 && p->ldi % 4 == 0 && p->q_off % 4 == 0 && p->k_off % 4 == 0 && p->v_off % 4 == 0 && p->ldq % 4 == 0 &&
                  p->ldk % 4 == 0 && p->ldv % 4 == 0 && al16(p->in) && al16(p->conv_state) && al16(p->conv_w) && al16(p->q_out) && al16(p->k_out) && al16(p->v_out) &&
                  (!p->channel_a || (al16(p->channel_a) && al16(p->channel_g) && al16(p->dt_bias)));
  DeltaArgs a{*p, N, vec, nullptr, 0, nullptr};
  const int units = 2 * p->kv_heads + p->heads + 1 + (p->channel_a ? p->heads : 0);
  const int longest = p->cu_seqlens ? std::min(N, std::max(max_qlen, 1)) : 1;
  NVC_REQUIRE(ctx, units <= 65535 && p->B <= 65535, NVC_ESHAPE, "more than 65 535 heads or sequences");
  const int warps = longest >= 4 ? 4 : 1;
  const dim3 grid((unsigned)((longest + warps - 1) / warps), units, p->B);
  auto* kernel = p->taps == 2 ? delta_prep_kernel<2> : (p->taps == 3 ? delta_prep_kernel<3> : (p->taps == 4 ? delta_prep_kernel<4> : delta_prep_kernel<0>));
  NVC_CUDA_CHECK(ctx, nvc_launch(ctx, kernel, grid, dim3(32 * warps), 0, nvc_stream(stream), a));
  ctx->launches++;
  return NVC_OK;
}

extern "C" int nvc_delta_rule_scan(nvc_ctx* ctx, const nvc_delta_prep* p, float* o, int ldo, float* state, int max_qlen, void* stream) {
  int rc = check_prep(ctx, p);
  if (rc) return rc;
  NVC_REQUIRE(ctx, o && state && ldo >= p->heads * p->vdim && max_qlen >= 1, NVC_EINVAL, "bad output / state");
  DeltaArgs a{*p, 0, 0, o, ldo, state};
  const int dim = p->dim;
  if (p->cu_seqlens && max_qlen >= 8 && dim <= 256) {
    // prompt portions: 16 tokens at a time (keys of more than 256 numbers stay token by token)
    auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
    a.vec = dim % 4 == 0 && p->ldq % 4 == 0 && p->ldk % 4 == 0 && al16(p->q_out) && al16(p->k_out) && al16(p->channel_g);
    const cudaError_t ce = p->channel_a ? launch_delta_chunk_sized<true>(ctx, a, nvc_stream(stream)) : launch_delta_chunk_sized<false>(ctx, a, nvc_stream(stream));
    NVC_CUDA_CHECK(ctx, ce);
    ctx->launches++;
    return NVC_OK;
  }
  // about four row groups per value column: four times the warps - and loads in flight - of one thread per whole column, at the price
  // of one shared-memory reduction of three numbers per token
  const int dpt = dim <= 64 ? 16 : (dim <= 128 ? 32 : (dim <= 256 ? 64 : 128));
  const int groups = (dim + dpt - 1) / dpt;
  const dim3 grid(p->B, p->heads, (p->vdim + 31) / 32), block(32 * groups);
  const size_t smem = ((size_t)(p->channel_a ? 6 : 4) * dim + (size_t)3 * groups * 32) * sizeof(float);
  cudaError_t ce;
  auto go = [&](auto ch) {
    constexpr bool CH = decltype(ch)::value;
    switch (dpt) {
      case 16: ce = nvc_launch(ctx, delta_scan_kernel<16, CH>, grid, block, smem, nvc_stream(stream), a); break;
      case 32: ce = nvc_launch(ctx, delta_scan_kernel<32, CH>, grid, block, smem, nvc_stream(stream), a); break;
      case 64: ce = nvc_launch(ctx, delta_scan_kernel<64, CH>, grid, block, smem, nvc_stream(stream), a); break;
      default: ce = nvc_launch(ctx, delta_scan_kernel<128, CH>, grid, block, smem, nvc_stream(stream), a); break;
    }
  };
  if (p->channel_a) go(std::true_type());
  else go(std::false_type());
  NVC_CUDA_CHECK(ctx, ce);
  ctx->launches++;
  return NVC_OK;
}
