// nvc_streams_norm: the row operation of models whose residual is several fp32 streams X_1 .. X_n instead of one (hyper-connections).
// One pass over a token's rows closes a sublayer and opens the next:
//   y    = c0 f(y0 + b0, w0) + c1 f(y1, w1)          what the sublayer left; f = identity or a weighted RMS norm over the width
//   X_t <- sum_s mix[s, t] X_s + out_w[t] y          every new stream from ALL the old ones
//   u    = sum_t in_w[t] X_t                         what the next sublayer reads (plain sum without in_w)
//   out  = u / sqrt(mean(u^2) + eps) * norm_w        in the storage format (u itself without norm_w)
// A thread owns columns: it holds the old streams of its columns in registers while it writes the new ones, so the update runs in place.
// Traffic: the streams once in and once out, the sublayer's outputs once, the normed row once.  Arithmetic is fp32, every sum has a fixed
// order.
#include "typed.cuh"

#include <algorithm>

namespace {

constexpr int kMaxStreams = 16;

struct StreamArgs {
  nvc_streams_args p;
  void* out;
  int H;
};

// sum over the CTA; part: 33 floats of shared memory; every thread gets the result
__device__ __forceinline__ float block_sum(float v, float* part) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) t += part[w];
  __syncthreads();
  return t;
}

template <int P> struct Pack;
template <> struct Pack<1> {
  float v[1];
  static __device__ __forceinline__ Pack load(const float* p) { return {{*p}}; }
  __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
  __device__ __forceinline__ void store(__nv_bfloat16* p) const { *p = __float2bfloat16_rn(v[0]); }
};
template <> struct Pack<4> {
  float v[4];
  static __device__ __forceinline__ Pack load(const float* p) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    return {{x.x, x.y, x.z, x.w}};
  }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
  __device__ __forceinline__ void store(__nv_bfloat16* p) const {
    uint2 u;
    u.x = pack_bf16(v[0], v[1]);
    u.y = pack_bf16(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = u;
  }
};

// NS: the number of streams (1 .. 4), or an upper bound of it.  P: numbers per access.
constexpr int stream_threads(int ns) { return ns <= 8 ? 512 : 256; }      // a thread holds 4 ns old numbers
template <typename T, int NS, int P>
__global__ void __launch_bounds__(stream_threads(NS)) streams_norm_kernel(const StreamArgs a) {
  extern __shared__ __align__(16) float sm[];          // [H]: u; behind it y0 + b0 and y1, each where it is normed
  __shared__ float part[33];
  __shared__ float cf[kMaxStreams * kMaxStreams + 2 * kMaxStreams];      // mix, out_w, in_w
  pdl_trigger();
  const nvc_streams_args& p = a.p;
  const int n = NS <= 4 ? NS : p.streams, H = a.H;
  for (int i = threadIdx.x; i < n * n; i += blockDim.x) cf[i] = p.mix ? __ldg(p.mix + i) : (i / n == i % n ? 1.f : 0.f);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    cf[n * n + i] = p.out_w ? __ldg(p.out_w + i) : 0.f;
    cf[n * n + n + i] = p.in_w ? __ldg(p.in_w + i) : 1.f;
  }
  pdl_wait();
  const int64_t src = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  const float* y0 = p.y0 ? p.y0 + src * p.ldy : nullptr;
  const float* y1 = p.y1 ? p.y1 + src * p.ldy : nullptr;
  const float* x = p.x_in + src * p.ldx_in;
  float* xo = p.x_out ? p.x_out + src * p.ldx_out : nullptr;
  float* us = sm;
  float* r0 = sm + H;
  float* r1 = r0 + (p.w0 ? H : 0);
  const int step = P * blockDim.x;
  float f0 = p.c0, f1 = p.c1;
  if (p.w0) {
    float ss = 0.f;
    for (int j = P * threadIdx.x; j < H; j += step) {
      Pack<P> v = Pack<P>::load(y0 + j);
      if (p.b0) {
        const Pack<P> b = Pack<P>::load(p.b0 + j);
#pragma unroll
        for (int e = 0; e < P; ++e) v.v[e] += b.v[e];
      }
      v.store(r0 + j);
#pragma unroll
      for (int e = 0; e < P; ++e) ss += v.v[e] * v.v[e];
    }
    f0 = p.c0 / sqrtf(block_sum(ss, part) / (float)H + p.eps);
  }
  if (p.w1) {
    float ss = 0.f;
    for (int j = P * threadIdx.x; j < H; j += step) {
      const Pack<P> v = Pack<P>::load(y1 + j);
      v.store(r1 + j);
#pragma unroll
      for (int e = 0; e < P; ++e) ss += v.v[e] * v.v[e];
    }
    f1 = p.c1 / sqrtf(block_sum(ss, part) / (float)H + p.eps);
  }
  __syncthreads();                                     // the coefficients have arrived
  float ss = 0.f;
  for (int j = P * threadIdx.x; j < H; j += step) {
    Pack<P> xs[NS];
#pragma unroll
    for (int s = 0; s < NS; ++s)
      if (s < n) xs[s] = Pack<P>::load(x + (int64_t)s * p.sx_in + j);
    float y[P];
#pragma unroll
    for (int e = 0; e < P; ++e) y[e] = 0.f;
    if (y0) {
      Pack<P> v = Pack<P>::load(p.w0 ? r0 + j : y0 + j);
      if (p.b0 && !p.w0) {
        const Pack<P> b = Pack<P>::load(p.b0 + j);
#pragma unroll
        for (int e = 0; e < P; ++e) v.v[e] += b.v[e];
      }
      if (p.w0) {
        const Pack<P> w = Pack<P>::load(p.w0 + j);
#pragma unroll
        for (int e = 0; e < P; ++e) y[e] = v.v[e] * f0 * w.v[e];
      } else {
#pragma unroll
        for (int e = 0; e < P; ++e) y[e] = v.v[e] * f0;
      }
    }
    if (y1) {
      const Pack<P> v = Pack<P>::load(p.w1 ? r1 + j : y1 + j);
      if (p.w1) {
        const Pack<P> w = Pack<P>::load(p.w1 + j);
#pragma unroll
        for (int e = 0; e < P; ++e) y[e] += v.v[e] * f1 * w.v[e];
      } else {
#pragma unroll
        for (int e = 0; e < P; ++e) y[e] += v.v[e] * f1;
      }
    }
    Pack<P> u;
#pragma unroll
    for (int e = 0; e < P; ++e) u.v[e] = 0.f;
#pragma unroll
    for (int t = 0; t < NS; ++t) {
      if (t < n) {
        Pack<P> z;
        if (y0 || y1) {
          const float ow = cf[n * n + t];
#pragma unroll
          for (int e = 0; e < P; ++e) z.v[e] = ow * y[e];
#pragma unroll
          for (int s = 0; s < NS; ++s) {
            if (s < n) {
              const float m = cf[s * n + t];
#pragma unroll
              for (int e = 0; e < P; ++e) z.v[e] = fmaf(m, xs[s].v[e], z.v[e]);
            }
          }
        } else {
          z = xs[t];                                   // no sublayer behind this pass: the streams stay
        }
        if (xo) z.store(xo + (int64_t)t * p.sx_out + j);
        const float iw = cf[n * n + n + t];
#pragma unroll
        for (int e = 0; e < P; ++e) u.v[e] = fmaf(iw, z.v[e], u.v[e]);
      }
    }
    u.store(us + j);
#pragma unroll
    for (int e = 0; e < P; ++e) ss += u.v[e] * u.v[e];
  }
  if (!a.out) return;
  T* out = reinterpret_cast<T*>(a.out) + (int64_t)blockIdx.x * p.ldo;
  float r = 1.f;
  if (p.norm_w) r = 1.0f / sqrtf(block_sum(ss, part) / (float)H + p.eps);
  for (int j = P * threadIdx.x; j < H; j += step) {    // a thread reads back what it wrote itself
    Pack<P> u = Pack<P>::load(us + j);
    if (p.norm_w) {
      const Pack<P> w = Pack<P>::load(p.norm_w + j);
#pragma unroll
      for (int e = 0; e < P; ++e) u.v[e] = u.v[e] * r * w.v[e];
    }
    u.store(out + j);
  }
}

template <typename T, int NS>
int launch_streams(nvc_ctx* ctx, const StreamArgs& a, bool vec, int N, size_t smem, void* stream) {
  static bool attr_set = false;
  if (!attr_set && smem > 48 * 1024) {
    NVC_CUDA_CHECK(ctx, cudaFuncSetAttribute(streams_norm_kernel<T, NS, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 3 * 16384 * 4));
    NVC_CUDA_CHECK(ctx, cudaFuncSetAttribute(streams_norm_kernel<T, NS, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 3 * 16384 * 4));
    attr_set = true;
  }
  const int units = vec ? (a.H + 3) / 4 : a.H;
  const int threads = std::min(stream_threads(NS), std::max(64, (units + 31) / 32 * 32));
  if (vec) NVC_CUDA_CHECK(ctx, nvc_launch(ctx, streams_norm_kernel<T, NS, 4>, dim3(N), dim3(threads), smem, nvc_stream(stream), a));
  else NVC_CUDA_CHECK(ctx, nvc_launch(ctx, streams_norm_kernel<T, NS, 1>, dim3(N), dim3(threads), smem, nvc_stream(stream), a));
  ctx->launches++;
  return NVC_OK;
}

}  // namespace

extern "C" int nvc_streams_norm(nvc_ctx* ctx, const nvc_streams_args* p, void* out, int out_dtype, int N, int H, void* stream) {
  NVC_REQUIRE(ctx, ctx && p && p->x_in, NVC_EINVAL, "null pointer");
  NVC_REQUIRE(ctx, p->streams >= 1 && p->streams <= kMaxStreams, NVC_ESHAPE, "1 to 16 streams");
  NVC_REQUIRE(ctx, N >= 0 && H > 0 && H <= 16384 && (!out || p->ldo >= H) && (!(p->y0 || p->y1) || p->ldy >= H), NVC_EINVAL,
              "bad sizes (rows of up to 16 384 numbers)");
  NVC_REQUIRE(ctx, (p->y0 || !(p->w0 || p->b0)) && (p->y1 || !p->w1) && (out || !p->norm_w), NVC_EINVAL, "a weight without its input or output");
  NVC_REQUIRE(ctx, !(p->y0 || p->y1) || (p->mix && p->out_w), NVC_EINVAL, "a sublayer's output needs mix and out_w");
  NVC_REQUIRE(ctx, !(p->rows && p->x_out), NVC_EINVAL, "a gathering call does not write the streams back");
  NVC_REQUIRE(ctx, p->sx_in >= 0 && (!p->x_out || (p->sx_out >= H && p->ldx_out >= (p->streams - 1) * p->sx_out + H)) &&
                       p->ldx_in >= (p->streams - 1) * p->sx_in + H && (p->x_out != p->x_in || (p->sx_out == p->sx_in && p->ldx_out == p->ldx_in)),
              NVC_EINVAL, "bad stream strides");
  if (N == 0) return NVC_OK;
  StreamArgs a{*p, out, H};
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = ((H | p->ldx_in | p->sx_in) & 3) == 0 && (!p->x_out || ((p->ldx_out | p->sx_out) & 3) == 0) && (!(p->y0 || p->y1) || (p->ldy & 3) == 0) &&
                   (!out || ((p->ldo & 3) == 0 && (reinterpret_cast<uintptr_t>(out) & (out_dtype == NVC_DT_F32 ? 15 : 7)) == 0)) && al16(p->x_in) &&
                   al16(p->x_out) && al16(p->y0) && al16(p->b0) && al16(p->w0) && al16(p->y1) && al16(p->w1) && al16(p->norm_w);
  const size_t smem = (size_t)H * (1 + (p->w0 ? 1 : 0) + (p->w1 ? 1 : 0)) * sizeof(float);
  NVC_DISPATCH_DT(out_dtype, T, {
    switch (p->streams) {
      case 1: return launch_streams<T, 1>(ctx, a, vec, N, smem, stream);
      case 2: return launch_streams<T, 2>(ctx, a, vec, N, smem, stream);
      case 3: return launch_streams<T, 3>(ctx, a, vec, N, smem, stream);
      case 4: return launch_streams<T, 4>(ctx, a, vec, N, smem, stream);
      default: return p->streams <= 8 ? launch_streams<T, 8>(ctx, a, vec, N, smem, stream) : launch_streams<T, 16>(ctx, a, vec, N, smem, stream);
    }
  });
  return NVC_OK;
}
