// nvc_short_conv_advance: the state of a short causal convolution after a step - every sequence's last taps - 1 inputs, with the bias of
// the projection that made them - written into its state slot (a portion shorter than that keeps the tail of what the slot held).  It
// runs behind the kernel that applies the convolution, which still reads the old state.
#include "typed.cuh"

namespace {

constexpr int kMaxTaps = 16;

// thread = (sequence, channel): reads the taps - 1 inputs that end the sequence so far, then writes them
__global__ void conv_advance_kernel(const nvc_short_conv cv, const float* __restrict__ in, int ldi, int off, const float* __restrict__ bias, int C,
                                    const int32_t* __restrict__ positions) {
  pdl_trigger();
  pdl_wait();
  const int keep = cv.taps - 1;
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (int64_t)cv.B * C) return;
  const int b = (int)(i / C), c = (int)(i % C);
  const int r0 = cv.cu_seqlens ? cv.cu_seqlens[b] : b;
  const int r1 = cv.cu_seqlens ? cv.cu_seqlens[b + 1] : b + 1;
  const int qlen = r1 - r0;
  const bool fresh = positions[r0] == 0;
  const float bc = bias ? __ldg(bias + c) : 0.f;
  float* st = cv.state + (int64_t)cv.state_slots[b] * keep * C;
  float v[kMaxTaps];
#pragma unroll
  for (int j = 0; j < kMaxTaps; ++j) {
    if (j < keep) {
      const int idx = qlen - keep + j;
      if (idx >= 0) v[j] = in[(int64_t)(r0 + idx) * ldi + off + c] + bc;
      else v[j] = fresh ? 0.f : st[(int64_t)(keep + idx) * C + c];
    }
  }
#pragma unroll
  for (int j = 0; j < kMaxTaps; ++j)
    if (j < keep) st[(int64_t)j * C + c] = v[j];
}

}  // namespace

extern "C" int nvc_short_conv_advance(nvc_ctx* ctx, const nvc_short_conv* cv, const float* in, int ldi, int off, const float* bias, int C,
                                      const int32_t* positions, void* stream) {
  NVC_REQUIRE(ctx, ctx && cv && cv->state && cv->state_slots && in && positions, NVC_EINVAL, "null pointer");
  NVC_REQUIRE(ctx, cv->taps >= 1 && cv->taps <= kMaxTaps && cv->B > 0 && C > 0 && off >= 0 && ldi >= off + C, NVC_EINVAL, "bad sizes (up to 16 taps)");
  if (cv->taps == 1) return NVC_OK;
  const int64_t total = (int64_t)cv->B * C;
  NVC_CUDA_CHECK(ctx, nvc_launch(ctx, conv_advance_kernel, dim3((unsigned)((total + 127) / 128)), dim3(128), 0, nvc_stream(stream), *cv, in, ldi, off,
                                 bias, C, positions));
  ctx->launches++;
  return NVC_OK;
}
