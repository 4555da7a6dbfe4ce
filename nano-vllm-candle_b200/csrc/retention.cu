// nvc_retention_scan: linear attention with a fixed decay per head and no softmax or denominator,
//   S_t = decay_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,
// over the new tokens of every sequence of a step, token by token.  The state S [dim, vdim] of every (sequence, head) lives in
// fp32 in a pool of state slots: a sequence whose first new token sits at position 0 starts from zeros, every other one from what
// its slot holds, and the slot is written back after the last token.  q, k, v, o are fp32 rows (the caller has already rotated q and
// k and scaled k).
//
// Two kernels, both with one CTA per (sequence, head, slice of value columns):
//   retention_scan_kernel    token by token (decode steps and very short portions), slices of 32 columns: thread (column v, row group r)
//                            keeps rows [r DPT, (r + 1) DPT) of column v of the state in registers (32 rows per warp, up to 32 warps);
//                            2 DPT FMAs per thread and token and, when the rows are split, one shared-memory reduction; the next
//                            token's q / k / v are fetched meanwhile.
//   retention_chunk_kernel   32 tokens at a time (prompt portions), slices of 32, 64 or 128 columns whose state stays in shared memory
//                            (every product is a tile of 8 rows or 4 rows x C columns per thread), the same recurrence regrouped:
//                              A[t][j] = decay^(t - j) (q_t . k_j), j <= t            inside the chunk
//                              o_t     = sum_j A[t][j] v_j + decay^(t + 1) S^T q_t     S: the state before the chunk
//                              S      <- decay^n S + sum_j decay^(n - 1 - j) k_j v_j^T n: tokens of the chunk
//                            Powers of the decay come from a table built by repeated multiplication (exact for 0 and 1).
// Both are plain fp32 FMA code; they differ from one another by rounding only.
//
// nvc_decay_scan is the same pair of kernels with what other linear recurrences of this shape need (kVar):
//   a decay per token and head, given as its logarithm: S_t = exp(l_t) S_(t-1) + k_t v_t^T.  Inside a chunk only differences of the
//     running sums L_t = l_0 + .. + l_t are exponentiated (all <= 0): A[t][j] carries exp(L_t - L_j), the state's share exp(L_t), the
//     state update exp(L_(n-1) - L_j); a decay that underflows stays a plain zero;
//   q and k heads shared by groups of value heads (head h reads q / k head h / (heads / qk_heads));
//   a skip term o_t += skip_w[h] * skip_t.
// nvc_memory_scan is the same pair of kernels for a matrix memory with an exponential input gate i_t and a forget gate f_t (logarithms),
// stabilised by a running maximum m_t = max(f_t + m_(t-1), i_t):
//   S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T,   n_t likewise with k_t alone,
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + eps)
//   Every CTA carries n and m itself; the slot holds a copy per 32 value columns, so that no slice waits for another.
//   Inside a chunk, with F_t the running sum of f and b_j = i_j - F_j:  M_t = max(m, b_0 .. b_t), m_t = F_t + M_t, and the decay of the
//   state up to token t is exp(m - M_t), the weight of token j at token t exp(b_j - M_t): every exponent is <= 0.  F, b and M are kept in
//   double precision (32 numbers per chunk), so a long run of small forget gates costs no digits of the differences.
//
// A selective state space layer in its dual form is the decayed recurrence with q = C, k = B, v = dt x, l = -exp(A_log) dt, skip = x.
#include "scan_common.cuh"

namespace {

struct RetArgs {
  const float *q, *k, *v;
  float* o;
  int ldq, ldk, ldv, ldo;
  float* state;                  // [slots, heads, dim, vdim]
  const int32_t *state_slots, *cu_seqlens, *positions;
  const float* decay;            // [heads]                       (kFixed)
  int heads, dim, vdim;
  int qk_heads;                  // q / k heads (a divisor of heads)
  const float* log_decay;        // [rows, ldl], one per head       (kVar)
  int ldl;
  const float* skip;             // [rows, lds] like v, or NULL
  const float* skip_w;           // [heads]
  int lds;
  nvc_memory_scan_args mem;      // gates, scale and state copies     (kMemory)
};

// what the recurrence is: a constant decay per head, a decay per token and head, the gated memory with its normaliser
enum Mode { kFixed, kVar, kMemory };

__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

template <int DPT, int MODE>
__global__ void retention_scan_kernel(const RetArgs a) {
  constexpr bool VAR = MODE == kVar, MEM = MODE == kMemory;
  static_assert(!MEM || DPT <= 32, "a lane keeps one number of n");
  extern __shared__ float sm[];
  pdl_trigger();
  const int b = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * 32;
  const int lane = threadIdx.x & 31, rg = threadIdx.x >> 5, groups = blockDim.x >> 5;
  const int v = v0 + lane;
  const bool vok = v < a.vdim;
  float* q_s = sm;                    // [2][dim]
  float* k_s = sm + 2 * a.dim;        // [2][dim]
  float* red = sm + 4 * a.dim;        // [groups][32]; MEM: behind it [groups], the shares of n . q
  float* red_n = red + groups * 32;
  const int hq = h / (a.heads / a.qk_heads);
  float dec = MODE == kFixed ? __ldg(a.decay + h) : 0.f;
  const float qs = MEM ? a.mem.q_scale : 1.f;
  const float sw = a.skip ? __ldg(a.skip_w + h) : 0.f;
  pdl_wait();
  const int r0 = a.cu_seqlens ? a.cu_seqlens[b] : b;
  const int r1 = a.cu_seqlens ? a.cu_seqlens[b + 1] : b + 1;
  const int d0 = rg * DPT;
  float S[DPT];
  float* sp = a.state + (((int64_t)a.state_slots[b] * a.heads + h) * a.dim) * a.vdim;
  const bool fresh = a.positions[r0] == 0;
#pragma unroll
  for (int i = 0; i < DPT; ++i) S[i] = (!fresh && vok && d0 + i < a.dim) ? sp[(int64_t)(d0 + i) * a.vdim + v] : 0.f;
  // MEM: this warp's rows of n, one per lane, and the running maximum
  float nk = 0.f, m = 0.f, zi = 0.f, zf = 0.f, bi = 0.f, bf = 0.f;
  const bool nok = MEM && lane < DPT && d0 + lane < a.dim;
  float* np = MEM ? a.mem.nm_state + (((int64_t)a.state_slots[b] * a.heads + h) * gridDim.z + blockIdx.z) * (a.dim + 1) : nullptr;
  if (MEM) {
    if (!fresh) { nk = nok ? np[d0 + lane] : 0.f; m = np[a.dim]; }
    zi = a.mem.i_in[(int64_t)r0 * a.mem.ldg + h];
    zf = a.mem.f_in[(int64_t)r0 * a.mem.ldg + h];
    bi = __ldg(a.mem.i_bias + h);
    bf = __ldg(a.mem.f_bias + h);
  }
  // stage token r0
  for (int d = threadIdx.x; d < a.dim; d += blockDim.x) {
    q_s[d] = MEM ? qs * a.q[(int64_t)r0 * a.ldq + hq * a.dim + d] : a.q[(int64_t)r0 * a.ldq + hq * a.dim + d];
    k_s[d] = a.k[(int64_t)r0 * a.ldk + hq * a.dim + d];
  }
  float vt = vok ? a.v[(int64_t)r0 * a.ldv + h * a.vdim + v] : 0.f;
  float ln = VAR ? a.log_decay[(int64_t)r0 * a.ldl + h] : 0.f;
  __syncthreads();
  for (int t = r0; t < r1; ++t) {
    const int cur = (t - r0) & 1;
    const float* qc = q_s + cur * a.dim;
    const float* kc = k_s + cur * a.dim;
    float vn = 0.f;
    if (t + 1 < r1) {       // fetch the next token into the other buffer
      for (int d = threadIdx.x; d < a.dim; d += blockDim.x) {
        q_s[(cur ^ 1) * a.dim + d] = MEM ? qs * a.q[(int64_t)(t + 1) * a.ldq + hq * a.dim + d] : a.q[(int64_t)(t + 1) * a.ldq + hq * a.dim + d];
        k_s[(cur ^ 1) * a.dim + d] = a.k[(int64_t)(t + 1) * a.ldk + hq * a.dim + d];
      }
      vn = vok ? a.v[(int64_t)(t + 1) * a.ldv + h * a.vdim + v] : 0.f;
    }
    if (VAR) {
      dec = expf(ln);
      if (t + 1 < r1) ln = a.log_decay[(int64_t)(t + 1) * a.ldl + h];
    }
    float nq = 0.f;
    if (MEM) {
      const float gi = capped(zi + bi, a.mem.cap), gf = log_sigmoid(capped(zf + bf, a.mem.cap));
      const float mt = fmaxf(gf + m, gi), add = expf(gi - mt);
      dec = expf(gf + m - mt);
      vt *= add;
      m = mt;
      if (nok) {
        nk = fmaf(dec, nk, add * kc[d0 + lane]);
        nq = nk * qc[d0 + lane];
      }
      nq = warp_sum(nq);
      if (t + 1 < r1) {
        zi = a.mem.i_in[(int64_t)(t + 1) * a.mem.ldg + h];
        zf = a.mem.f_in[(int64_t)(t + 1) * a.mem.ldg + h];
      }
    }
    const float sk = (a.skip && vok) ? sw * a.skip[(int64_t)t * a.lds + h * a.vdim + v] : 0.f;
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
      if (d0 + i < a.dim) {
        S[i] = fmaf(dec, S[i], kc[d0 + i] * vt);
        acc = fmaf(S[i], qc[d0 + i], acc);
      }
    }
    if (groups > 1) {
      red[rg * 32 + lane] = acc;
      if (MEM && lane == 0) red_n[rg] = nq;
      __syncthreads();
      if (rg == 0) {
        float s = 0.f;
        for (int g = 0; g < groups; ++g) s += red[g * 32 + lane];
        if (MEM) {
          nq = 0.f;
          for (int g = 0; g < groups; ++g) nq += red_n[g];
          s = s / (fmaxf(fabsf(nq), expf(-m)) + a.mem.den_eps);
        }
        if (vok) a.o[(int64_t)t * a.ldo + h * a.vdim + v] = s + sk;
      }
    } else if (vok) {
      if (MEM) acc = acc / (fmaxf(fabsf(nq), expf(-m)) + a.mem.den_eps);
      a.o[(int64_t)t * a.ldo + h * a.vdim + v] = acc + sk;
    }
    vt = vn;
    __syncthreads();
  }
  if (vok)
#pragma unroll
    for (int i = 0; i < DPT; ++i)
      if (d0 + i < a.dim) sp[(int64_t)(d0 + i) * a.vdim + v] = S[i];
  if (nok) np[d0 + lane] = nk;
  if (MEM && threadIdx.x == 0) np[a.dim] = m;
}

constexpr int kChunk = 32;          // tokens per chunk
constexpr int kChunkA = kChunk + 4; // row stride of A (16-byte rows)

// shared memory of a CTA: q and k of the chunk, A, the state's columns, the gate arrays of the chunk
__host__ __device__ inline size_t chunk_smem_floats(int dim, int cols) {
  const int dz = scan_row(dim);
  return (size_t)2 * kChunk * (dz + 4) + kChunk * kChunkA + (size_t)dz * cols + dz + 4 * kChunk + 4 * kChunk + kChunk + 4;
}

// One CTA per (sequence, head, COLS = 32 C NW / 4 value columns); its slice of the state stays in shared memory.  Stages of a chunk:
//   copy      q and k, asynchronously; the chunk's decays or gates by one warp
//   products  A, rows t against eight earlier tokens at a time, lanes along the channels (scan_common.cuh)
//   state     a warp takes 8 of the 32 queries against 32 C columns of the state: 8 C sums per thread
//   outputs   A against the values (straight from global memory, 32 C numbers per thread), then the state update 4 rows at a time
template <int C, int NW, int MODE>
__global__ void __launch_bounds__(NW * 32, 2) retention_chunk_kernel(const RetArgs a, const int vec) {
  constexpr bool VAR = MODE == kVar, MEM = MODE == kMemory;
  constexpr int COLS = 32 * C * (NW / 4), THREADS = NW * 32;
  extern __shared__ __align__(16) float sm[];
  pdl_trigger();
  const int b = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * COLS;
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, rg = w & 3;
  const int dim = a.dim, dz = scan_row(dim), ds = dz + 4;
  float* Qs = sm;                          // [32][ds]
  float* Ks = Qs + kChunk * ds;            // [32][ds]
  float* As = Ks + kChunk * ds;            // [32][36]  A[t][j], zero above the diagonal
  float* Ss = As + kChunk * kChunkA;       // [dz][COLS]
  float* n_s = Ss + (size_t)dz * COLS;     // [dz] MEM: n, zeros behind dim
  double* bD = reinterpret_cast<double*>(n_s + dz);        // [32] MEM: b_j = i_j - F_j
  double* MD = bD + kChunk;                                // [32] MEM: M_t
  float* keep_s = reinterpret_cast<float*>(MD + kChunk);   // [32] the state's decay up to token t
  float* wj_s = keep_s + kChunk;                           // [32] the weight of token j in the state behind the chunk
  float* em_s = wj_s + kChunk;                             // [32] MEM: exp(-m_t)
  float* nq_s = em_s + kChunk;                             // [32] MEM: n . q_t
  float* gp = nq_s + kChunk;                               // [33] decay^0 .. decay^32;  VAR: the running sums L_0 .. L_31
  double m0 = 0.0;                                         // MEM, warp 0: the running maximum in front of the chunk
  const int hq = h / (a.heads / a.qk_heads);
  const float sw = a.skip ? __ldg(a.skip_w + h) : 0.f;
  const float qs = MEM ? a.mem.q_scale : 1.f;
  if (MODE == kFixed && threadIdx.x == 0) {
    const float dec = __ldg(a.decay + h);
    float p = 1.f;
    for (int i = 0; i <= kChunk; ++i) { gp[i] = p; p *= dec; }
  }
  pdl_wait();
  const int r0 = a.cu_seqlens ? a.cu_seqlens[b] : b;
  const int r1 = a.cu_seqlens ? a.cu_seqlens[b + 1] : b + 1;
  const int slot = a.state_slots[b];
  const bool fresh = a.positions[r0] == 0;
  float* sp = a.state + (((int64_t)slot * a.heads + h) * dim) * a.vdim;
  for (int i = threadIdx.x; i < dz * COLS; i += THREADS) {
    const int d = i / COLS, c = i % COLS;
    Ss[i] = (!fresh && d < dim && v0 + c < a.vdim) ? sp[(int64_t)d * a.vdim + v0 + c] : 0.f;
  }
  for (int i = threadIdx.x; i < kChunk * kChunkA; i += THREADS) As[i] = 0.f;      // what the products never write stays zero
  // MEM: n and m of this CTA's columns; a copy per 32 of them, all alike
  const int copies = (a.vdim + 31) / 32;
  float* np = MEM ? a.mem.nm_state + (((int64_t)slot * a.heads + h) * copies + v0 / 32) * (dim + 1) : nullptr;
  if (MEM) {
    for (int d = threadIdx.x; d < dz; d += THREADS) n_s[d] = (!fresh && d < dim) ? np[d] : 0.f;
    if (!fresh) m0 = (double)np[dim];
  }
  const int cl = (w >> 2) * 32 * C + lane * C;             // this lane's first column of the slice
  for (int c0 = r0; c0 < r1; c0 += kChunk) {
    const int n = min(kChunk, r1 - c0);
    __syncthreads();                                       // the previous chunk is done with the staged rows
    for (int t = w; t < kChunk; t += NW) {
      copy_row(Qs + t * ds, a.q + (int64_t)(c0 + t) * a.ldq + hq * dim, dim, dz, t < n, vec, lane);
      copy_row(Ks + t * ds, a.k + (int64_t)(c0 + t) * a.ldk + hq * dim, dim, dz, t < n, vec, lane);
    }
    if (w == 0) {
      if (MODE == kFixed) {
        keep_s[lane] = gp[min(lane, n - 1) + 1];
        wj_s[lane] = lane < n ? gp[n - 1 - lane] : 0.f;
      } else if (VAR) {       // inclusive running sums of the chunk's log decays (a fixed order: lane by lane)
        float l = lane < n ? a.log_decay[(int64_t)(c0 + lane) * a.ldl + h] : 0.f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float up = __shfl_up_sync(0xffffffffu, l, o);
          if (lane >= o) l += up;
        }
        gp[lane] = l;
        keep_s[lane] = expf(l);
        wj_s[lane] = expf(__shfl_sync(0xffffffffu, l, n - 1) - l);
      } else {
        const bool in = lane < n;
        const int64_t gr = (int64_t)(c0 + lane) * a.mem.ldg + h;
        const float gi = in ? capped(a.mem.i_in[gr] + __ldg(a.mem.i_bias + h), a.mem.cap) : -INFINITY;      // no token: weight 0
        double F = in ? (double)log_sigmoid(capped(a.mem.f_in[gr] + __ldg(a.mem.f_bias + h), a.mem.cap)) : 0.0;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const double up = __shfl_up_sync(0xffffffffu, F, o);
          if (lane >= o) F += up;
        }
        const double bj = (double)gi - F;
        double M = fmax(bj, m0);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const double up = __shfl_up_sync(0xffffffffu, M, o);
          if (lane >= o) M = fmax(M, up);
        }
        const double Mn = __shfl_sync(0xffffffffu, M, n - 1), Fn = __shfl_sync(0xffffffffu, F, n - 1);
        bD[lane] = bj;
        MD[lane] = M;
        keep_s[lane] = expf((float)(m0 - M));
        em_s[lane] = expf((float)-(F + M));
        wj_s[lane] = expf((float)(bj - Mn));
        m0 = Fn + Mn;
      }
    }
    copy_async_wait();
    __syncthreads();
    // ---- A[t][j]: a row t against eight earlier tokens at a time, groups of GL lanes along the channels
    {
      const int GL = dz > 64 ? 32 : (dz > 32 ? 16 : 8), gl = lane & (GL - 1), sub = lane / GL, subs = 32 / GL;
#pragma unroll 1
      for (int i = 0; i < kChunk / NW; ++i) {               // rows in pairs that add up to equal work
        const int t = (i & 1) ? (i + 1) * NW - 1 - w : i * NW + w;
        const float* qt = Qs + t * ds;
        if (MEM) {
          float x = 0.f;
          for (int c = 4 * lane; c < dz; c += 128)
            x = fma4(*reinterpret_cast<const float4*>(qt + c), *reinterpret_cast<const float4*>(n_s + c), x);
          x = warp_sum(x);
          if (lane == 0) nq_s[t] = qs * x;
        }
#pragma unroll 1
        for (int j0 = 0; j0 <= t; j0 += 8 * subs) {
          const int jb = min(j0 + 8 * sub, kChunk - 8);     // groups behind the last row repeat it
          float v[8];
#pragma unroll
          for (int y = 0; y < 8; ++y) v[y] = 0.f;
          for (int c = 4 * gl; c < dz; c += 4 * GL) {
            const float4 x = *reinterpret_cast<const float4*>(qt + c);
#pragma unroll
            for (int y = 0; y < 8; ++y) v[y] = fma4(x, *reinterpret_cast<const float4*>(Ks + (jb + y) * ds + c), v[y]);
          }
          int which;
          bool writer;
          const float sum = group_sum8(v, GL, gl, &which, &writer);
          const int j = jb + which;
          if (writer && j <= t) {
            const float f = MEM ? qs * expf((float)(bD[j] - MD[t])) : (VAR ? expf(gp[t] - gp[j]) : gp[t - j]);
            As[t * kChunkA + j] = f * sum;
          }
        }
      }
    }
    // ---- the state's share of every output: 8 queries per warp
    float acc[8][C];
#pragma unroll
    for (int r = 0; r < 8; ++r)
#pragma unroll
      for (int e = 0; e < C; ++e) acc[r][e] = 0.f;
    {
      const float* X = Qs + 8 * rg * ds;
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
    // the chunk's values of this lane's columns
    float vv[kChunk][C];
    {
      const float* vp = a.v + (int64_t)c0 * a.ldv + h * a.vdim + v0 + cl;
#pragma unroll
      for (int j = 0; j < kChunk; ++j)
#pragma unroll
        for (int e = 0; e < C; ++e) vv[j][e] = (j < n && v0 + cl + e < a.vdim) ? vp[(int64_t)j * a.ldv + e] : 0.f;
    }
    __syncthreads();                                       // A is complete, the state has been read
    // ---- outputs
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      const int t = 8 * rg + r;
      const float keep = keep_s[t] * qs;
      float o[C], den = 0.f;
#pragma unroll
      for (int e = 0; e < C; ++e) o[e] = keep * acc[r][e];
#pragma unroll
      for (int j4 = 0; j4 < kChunk; j4 += 4) {              // entries behind the diagonal are zero
        const float4 m = *reinterpret_cast<const float4*>(As + t * kChunkA + j4);
        if (MEM) den += (m.x + m.y) + (m.z + m.w);
#pragma unroll
        for (int e = 0; e < C; ++e) {
          o[e] = fmaf(m.x, vv[j4][e], o[e]);
          o[e] = fmaf(m.y, vv[j4 + 1][e], o[e]);
          o[e] = fmaf(m.z, vv[j4 + 2][e], o[e]);
          o[e] = fmaf(m.w, vv[j4 + 3][e], o[e]);
        }
      }
      if (MEM) {
        den = fmaxf(fabsf(fmaf(keep_s[t], nq_s[t], den)), em_s[t]) + a.mem.den_eps;
#pragma unroll
        for (int e = 0; e < C; ++e) o[e] /= den;
      }
      float* op = a.o + (int64_t)(c0 + t) * a.ldo + h * a.vdim + v0 + cl;
#pragma unroll
      for (int e = 0; e < C; ++e) {
        if (t < n && v0 + cl + e < a.vdim) {
          if (a.skip) o[e] += sw * a.skip[(int64_t)(c0 + t) * a.lds + h * a.vdim + v0 + cl + e];
          op[e] = o[e];
        }
      }
    }
    // ---- the state behind the chunk
    const float gn = keep_s[n - 1];
#pragma unroll
    for (int j = 0; j < kChunk; ++j) {
      const float f = wj_s[j];
#pragma unroll
      for (int e = 0; e < C; ++e) vv[j][e] *= f;
    }
    for (int d = 4 * rg; d < dz; d += 16) {
      float s[4][C];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        ld_cols<C>(s[i], Ss + (d + i) * COLS + cl);
#pragma unroll
        for (int e = 0; e < C; ++e) s[i][e] *= gn;
      }
#pragma unroll
      for (int j = 0; j < kChunk; ++j) {
        const float4 k = *reinterpret_cast<const float4*>(Ks + j * ds + d);
#pragma unroll
        for (int e = 0; e < C; ++e) {
          s[0][e] = fmaf(k.x, vv[j][e], s[0][e]);
          s[1][e] = fmaf(k.y, vv[j][e], s[1][e]);
          s[2][e] = fmaf(k.z, vv[j][e], s[2][e]);
          s[3][e] = fmaf(k.w, vv[j][e], s[3][e]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) st_cols<C>(Ss + (d + i) * COLS + cl, s[i]);
    }
    if (MEM) {
      for (int d = threadIdx.x; d < dim; d += THREADS) {
        float x = gn * n_s[d];
        for (int j = 0; j < n; ++j) x = fmaf(wj_s[j], Ks[j * ds + d], x);
        n_s[d] = x;                                        // read again behind the next chunk's first barrier
      }
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < dim * COLS; i += THREADS) {
    const int d = i / COLS, c = i % COLS;
    if (v0 + c < a.vdim) sp[(int64_t)d * a.vdim + v0 + c] = Ss[i];
  }
  if (MEM) {
    const int mine = min(COLS, a.vdim - v0), groups = (mine + 31) / 32;
    for (int g = 0; g < groups; ++g) {
      for (int d = threadIdx.x; d < dim; d += THREADS) np[(int64_t)g * (dim + 1) + d] = n_s[d];
      if (threadIdx.x == 0) np[(int64_t)g * (dim + 1) + dim] = (float)m0;
    }
  }
}

template <int C, int NW, int MODE>
cudaError_t launch_chunk(nvc_ctx* ctx, const RetArgs& a, int B, cudaStream_t st) {
  constexpr int COLS = 32 * C * (NW / 4);
  const size_t smem = chunk_smem_floats(a.dim, COLS) * sizeof(float);
  static bool attr_set = false;
  if (!attr_set && smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(retention_chunk_kernel<C, NW, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) return e;
    attr_set = true;
  }
  const int vec = (a.dim & 3) == 0 && (a.ldq & 3) == 0 && (a.ldk & 3) == 0 && ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.k)) & 15) == 0;
  return nvc_launch(ctx, retention_chunk_kernel<C, NW, MODE>, dim3(B, a.heads, (a.vdim + COLS - 1) / COLS), dim3(NW * 32), smem, st, a, vec);
}

template <int MODE>
int run_scan(nvc_ctx* ctx, const RetArgs& a, int B, int max_qlen, void* stream) {
  const int heads = a.heads, dim = a.dim, vdim = a.vdim;
  if (a.cu_seqlens && max_qlen > 4 && dim <= 512) {
    // prompt portions: 32 tokens at a time
    // wide slices while they fill the GPU; keys of more than 256 numbers leave room for 32 columns only
    cudaError_t ce;
    if (dim > 256) ce = launch_chunk<1, 4, MODE>(ctx, a, B, nvc_stream(stream));
    else if (vdim > 64 && 4 * B * heads * ((vdim + 127) / 128) >= 3 * ctx->num_sms) ce = launch_chunk<2, 8, MODE>(ctx, a, B, nvc_stream(stream));
    else ce = launch_chunk<1, 8, MODE>(ctx, a, B, nvc_stream(stream));
    NVC_CUDA_CHECK(ctx, ce);
    ctx->launches++;
    return NVC_OK;
  }
  // rows of a state column are split over warps of the CTA, 32 (16) rows each: a decode step is bound by reading and writing the
  // state once, and a CTA of one warp holding whole columns of 128 numbers leaves too few loads in flight
  const int dpt = dim <= 16 ? 16 : 32;
  const int groups = (dim + dpt - 1) / dpt;
  const dim3 grid(B, heads, (vdim + 31) / 32), block(32 * groups);
  const size_t smem = ((size_t)4 * dim + (size_t)groups * 33) * sizeof(float);
  cudaError_t ce;
  if (dpt == 16) ce = nvc_launch(ctx, retention_scan_kernel<16, MODE>, grid, block, smem, nvc_stream(stream), a);
  else ce = nvc_launch(ctx, retention_scan_kernel<32, MODE>, grid, block, smem, nvc_stream(stream), a);
  NVC_CUDA_CHECK(ctx, ce);
  ctx->launches++;
  return NVC_OK;
}

}  // namespace

extern "C" int nvc_retention_scan(nvc_ctx* ctx, const float* q, int ldq, const float* k, int ldk, const float* v, int ldv, float* o, int ldo,
                                  float* state, const int32_t* state_slots, const int32_t* cu_seqlens, const int32_t* positions,
                                  const float* decay, int B, int max_qlen, int heads, int dim, int vdim, void* stream) {
  NVC_REQUIRE(ctx, ctx && q && k && v && o && state && state_slots && positions && decay, NVC_EINVAL, "null pointer");
  NVC_REQUIRE(ctx, B > 0 && heads > 0 && dim > 0 && vdim > 0 && dim <= 1024 && heads <= 65535, NVC_EINVAL, "bad sizes");
  NVC_REQUIRE(ctx, ldq >= heads * dim && ldk >= heads * dim && ldv >= heads * vdim && ldo >= heads * vdim, NVC_EINVAL, "bad strides");
  RetArgs a{q, k, v, o, ldq, ldk, ldv, ldo, state, state_slots, cu_seqlens, positions, decay, heads, dim, vdim, heads, nullptr, 0, nullptr, nullptr, 0, {}};
  return run_scan<kFixed>(ctx, a, B, max_qlen, stream);
}

extern "C" int nvc_decay_scan(nvc_ctx* ctx, const nvc_decay_scan_args* p, int B, int max_qlen, void* stream) {
  NVC_REQUIRE(ctx, ctx && p && p->q && p->k && p->v && p->o && p->state && p->state_slots && p->positions, NVC_EINVAL, "null pointer");
  NVC_REQUIRE(ctx, (p->decay != nullptr) != (p->log_decay != nullptr), NVC_EINVAL, "one of decay and log_decay");
  NVC_REQUIRE(ctx, B > 0 && p->heads > 0 && p->qk_heads > 0 && p->heads % p->qk_heads == 0 && p->dim > 0 && p->vdim > 0 && p->dim <= 1024 &&
                       p->heads <= 65535,
              NVC_EINVAL, "bad sizes");
  NVC_REQUIRE(ctx, p->ldq >= p->qk_heads * p->dim && p->ldk >= p->qk_heads * p->dim && p->ldv >= p->heads * p->vdim && p->ldo >= p->heads * p->vdim &&
                       (!p->log_decay || p->ldl >= p->heads) && (!p->skip || (p->skip_w && p->lds >= p->heads * p->vdim)),
              NVC_EINVAL, "bad strides");
  RetArgs a{p->q, p->k, p->v, p->o, p->ldq, p->ldk, p->ldv, p->ldo, p->state, p->state_slots, p->cu_seqlens, p->positions, p->decay,
            p->heads, p->dim, p->vdim, p->qk_heads, p->log_decay, p->ldl, p->skip, p->skip_w, p->lds, {}};
  return p->log_decay ? run_scan<kVar>(ctx, a, B, max_qlen, stream) : run_scan<kFixed>(ctx, a, B, max_qlen, stream);
}

extern "C" int nvc_memory_scan(nvc_ctx* ctx, const nvc_memory_scan_args* p, int B, int max_qlen, void* stream) {
  NVC_REQUIRE(ctx, ctx && p && p->q && p->k && p->v && p->i_in && p->f_in && p->i_bias && p->f_bias && p->o && p->state && p->nm_state && p->state_slots &&
                       p->positions,
              NVC_EINVAL, "null pointer");
  NVC_REQUIRE(ctx, B > 0 && p->heads > 0 && p->dim > 0 && p->vdim > 0 && p->dim <= 1024 && p->heads <= 65535 && p->cap > 0.f, NVC_EINVAL, "bad sizes");
  NVC_REQUIRE(ctx, p->ldq >= p->heads * p->dim && p->ldk >= p->heads * p->dim && p->ldv >= p->heads * p->vdim && p->ldo >= p->heads * p->vdim &&
                       p->ldg >= p->heads,
              NVC_EINVAL, "bad strides");
  RetArgs a{p->q, p->k, p->v, p->o, p->ldq, p->ldk, p->ldv, p->ldo, p->state, p->state_slots, p->cu_seqlens, p->positions, nullptr,
            p->heads, p->dim, p->vdim, p->heads, nullptr, 0, nullptr, nullptr, 0, *p};
  return run_scan<kMemory>(ctx, a, B, max_qlen, stream);
}
