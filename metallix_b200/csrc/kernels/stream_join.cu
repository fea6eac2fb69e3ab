// What a product over [x; x0] reads, where x is the residual stream (with a
// sublayer's result still to be added) and x0 the stream as the embedding left
// it: out[t] = [x[t] + delta[t] | x0[t]] in the compute type, the sum in
// float32, one rounding. The product's result is a new stream, so x itself is
// left as it is. Four values a thread.
#include "common.cuh"

namespace mxb {

__device__ __forceinline__ float4 join_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 join_load4(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(raw.x << 16), __uint_as_float(raw.x & 0xffff0000u),
                     __uint_as_float(raw.y << 16), __uint_as_float(raw.y & 0xffff0000u));
}
__device__ __forceinline__ void join_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void join_store4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
}

template <typename TDelta, typename TOut>
__global__ void __launch_bounds__(256)
join_rows_kernel(const float* __restrict__ x, const TDelta* __restrict__ delta, const float* __restrict__ first,
                 TOut* __restrict__ out, int width, long long groups) {
  chain_release();
  chain_wait();
  const long long index = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (index >= groups) return;
  const int per_row = width / 4;
  const long long t = index / per_row;
  const int c = static_cast<int>(index - t * per_row) * 4;
  float4 v = join_load4(behind_wait(x) + t * width + c);
  if (delta != nullptr) {
    const float4 d = join_load4(behind_wait(delta) + t * width + c);
    v.x += d.x; v.y += d.y; v.z += d.z; v.w += d.w;
  }
  TOut* row = out + t * 2 * width;
  join_store4(row + c, v);
  join_store4(row + width + c, join_load4(behind_wait(first) + t * width + c));
}

}  // namespace mxb

using namespace mxb;

// x, first: float32 [tokens, width]; delta: [tokens, width] of delta_dtype, or null; out: [tokens, 2 * width].
// width a multiple of 8, everything 16-byte aligned.
MXB_API int mxb_join_rows(const float* x, const void* delta, int delta_dtype, const float* first, void* out, int out_dtype,
                          int tokens, int width, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  if (width <= 0 || width % 8 != 0 || !aligned(x) || !aligned(delta) || !aligned(first) || !aligned(out))
    return static_cast<int>(cudaErrorInvalidValue);
  const long long groups = static_cast<long long>(tokens) * (width / 4);
  const unsigned blocks = static_cast<unsigned>((groups + 255) / 256);
#define GO(TD, TO)                                                                                              \
  return static_cast<int>(launch_chained(join_rows_kernel<TD, TO>, dim3(blocks), dim3(256), 0, stream, x,       \
                                         static_cast<const TD*>(delta), first, static_cast<TO*>(out), width, groups))
  if (delta == nullptr || delta_dtype == kF32) {
    if (out_dtype == kF32) GO(float, float);
    if (out_dtype == kBF16) GO(float, __nv_bfloat16);
  } else if (delta_dtype == kBF16) {
    if (out_dtype == kF32) GO(__nv_bfloat16, float);
    if (out_dtype == kBF16) GO(__nv_bfloat16, __nv_bfloat16);
  }
#undef GO
  return static_cast<int>(cudaErrorInvalidValue);
}
