// What the chunked recurrences (delta_rule.cu, retention.cu) share: asynchronous copies of fp32 rows into shared memory, sums over groups of
// lanes by exchange, a thread's C neighbouring columns.
#pragma once
#include "typed.cuh"

namespace {

__device__ __forceinline__ float ex2(float x) {          // 2^x
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void copy_async16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_async4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_async_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

__device__ __forceinline__ float fma4(const float4& x, const float4& y, float acc) {
  acc = fmaf(x.x, y.x, acc);
  acc = fmaf(x.y, y.y, acc);
  acc = fmaf(x.z, y.z, acc);
  return fmaf(x.w, y.w, acc);
}

template <int C> __device__ __forceinline__ void ld_cols(float (&x)[C], const float* p) {
  if constexpr (C == 2) { const float2 v = *reinterpret_cast<const float2*>(p); x[0] = v.x; x[1] = v.y; }
  else x[0] = *p;
}
template <int C> __device__ __forceinline__ void st_cols(float* p, const float (&x)[C]) {
  if constexpr (C == 2) *reinterpret_cast<float2*>(p) = make_float2(x[0], x[1]);
  else *p = x[0];
}

__host__ __device__ inline int scan_row(int dim) { return (dim + 7) / 8 * 8; }       // staged numbers of a row (zeros behind dim)

// One row of `dim` numbers into shared memory, zeros from there to dz (in == false: zeros everywhere).  vec: dim is a multiple of 4 and the
// source 16-byte aligned.  One warp; wait with copy_async_wait and a barrier.
__device__ __forceinline__ void copy_row(float* dst, const float* src, int dim, int dz, bool in, bool vec, int lane) {
  if (vec && in) {
    for (int c = 4 * lane; c < dz; c += 128) {
      if (c < dim) copy_async16(dst + c, src + c);
      else *reinterpret_cast<float4*>(dst + c) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
  } else {
    for (int c = lane; c < dz; c += 32) {
      if (in && c < dim) copy_async4(dst + c, src + c);
      else dst[c] = 0.f;
    }
  }
}

// Eight sums of a group of GL (8, 16 or 32) lanes at once: with every step a lane keeps half of its sums and one more bit of which ones.
// Returns the sum number `which` in the lanes where *writer is set.
__device__ __forceinline__ float group_sum8(float (&v)[8], int GL, int gl, int* which, bool* writer) {
  int o = GL >> 1, id = 0;
#pragma unroll
  for (int half = 4; half > 0; half >>= 1, o >>= 1) {
    const bool up = (gl & o) != 0;
#pragma unroll
    for (int y = 0; y < half; ++y) {
      const float give = up ? v[y] : v[y + half], keep = up ? v[y + half] : v[y];
      v[y] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
    id = 2 * id + (up ? 1 : 0);
  }
  for (; o > 0; o >>= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
  *which = id;
  *writer = (gl & (GL / 8 - 1)) == 0;
  return v[0];
}

}  // namespace
