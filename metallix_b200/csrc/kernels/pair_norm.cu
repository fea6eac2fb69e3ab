// Two mixers side by side whose outputs each pass an RMS norm of their own
// before they join the residual stream, and the next sublayer's norm, in one
// pass over the row:
//
//   l = left (+ left_bias),   r = right (+ right_bias)
//   x += a * l * rsqrt(mean(l^2) + left_eps) * wl + b * r * rsqrt(mean(r^2) + right_eps) * wr
//   y = x * rsqrt(mean(x^2) + eps) * w                       (y optional)
//
// All of it float32. `left` may be a sum its producer left in parts, float32
// [parts, rows, size], which are added up in their order first (the output
// projection of a decode step's attention, taken head by head). One block per
// row, four values a thread at a time; both rows wait in shared memory
// between the passes, each value read only by the thread that put it there.
#include "common.cuh"

namespace mxb {

constexpr int kPairThreads = 256;

__device__ __forceinline__ float4 pair_load4(const void* p, int code, size_t index) {
  if (code == kF32) return *reinterpret_cast<const float4*>(static_cast<const float*>(p) + index);
  const uint2 raw = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p) + index);
  return make_float4(__uint_as_float(raw.x << 16), __uint_as_float(raw.x & 0xffff0000u),
                     __uint_as_float(raw.y << 16), __uint_as_float(raw.y & 0xffff0000u));
}
__device__ __forceinline__ void pair_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void pair_store4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
}
__device__ __forceinline__ float4 pair_sum(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float pair_square(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// Two sums over the block at once; every thread gets both.
__device__ __forceinline__ float2 pair_block_sums(float a, float b, float2* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  if (lane == 0) scratch[warp] = make_float2(a, b);
  __syncthreads();
  float2 total = make_float2(0.0f, 0.0f);
  for (int i = 0; i < warps; ++i) {   // warp order: one order of additions
    total.x += scratch[i].x;
    total.y += scratch[i].y;
  }
  return total;
}

template <typename TOut>
__global__ void __launch_bounds__(kPairThreads)
pair_norm_kernel(float* __restrict__ x, const void* __restrict__ left, int left_code, int left_parts,
                 const void* __restrict__ right, int right_code, const float* __restrict__ left_bias,
                 const float* __restrict__ right_bias, const float* __restrict__ wl, const float* __restrict__ wr,
                 float left_eps, float right_eps, float a, float b, TOut* __restrict__ y, const float* __restrict__ w,
                 int rows, int size, float eps) {
  extern __shared__ __align__(16) float pair_rows[];   // the left row, then the right one
  __shared__ float2 scratch[kPairThreads / 32];
  __shared__ float scratch_one[33];
  float* s_left = pair_rows;
  float* s_right = pair_rows + size;
  chain_release();
  const size_t base = static_cast<size_t>(blockIdx.x) * size;
  chain_wait();
  float* row = behind_wait(x) + base;
  left = behind_wait(left);
  right = behind_wait(right);
  float sum_left = 0.0f, sum_right = 0.0f;
  for (int i = threadIdx.x * 4; i < size; i += blockDim.x * 4) {
    float4 l = pair_load4(left, left_code, base + i);
    for (int part = 1; part < left_parts; ++part)
      l = pair_sum(l, pair_load4(left, left_code, static_cast<size_t>(part) * rows * size + base + i));
    if (left_bias != nullptr) l = pair_sum(l, *reinterpret_cast<const float4*>(left_bias + i));
    float4 r = pair_load4(right, right_code, base + i);
    if (right_bias != nullptr) r = pair_sum(r, *reinterpret_cast<const float4*>(right_bias + i));
    sum_left += pair_square(l);
    sum_right += pair_square(r);
    pair_store4(s_left + i, l);
    pair_store4(s_right + i, r);
  }
  const float2 sums = pair_block_sums(sum_left, sum_right, scratch);
  const float scale_left = a * rsqrtf(sums.x / static_cast<float>(size) + left_eps);
  const float scale_right = b * rsqrtf(sums.y / static_cast<float>(size) + right_eps);
  float sum = 0.0f;
  for (int i = threadIdx.x * 4; i < size; i += blockDim.x * 4) {
    const float4 l = *reinterpret_cast<const float4*>(s_left + i), r = *reinterpret_cast<const float4*>(s_right + i);
    const float4 gl = *reinterpret_cast<const float4*>(wl + i), gr = *reinterpret_cast<const float4*>(wr + i);
    float4 v = *reinterpret_cast<const float4*>(row + i);
    v.x += l.x * scale_left * gl.x + r.x * scale_right * gr.x;
    v.y += l.y * scale_left * gl.y + r.y * scale_right * gr.y;
    v.z += l.z * scale_left * gl.z + r.z * scale_right * gr.z;
    v.w += l.w * scale_left * gl.w + r.w * scale_right * gr.w;
    *reinterpret_cast<float4*>(row + i) = v;
    pair_store4(s_left + i, v);
    sum += pair_square(v);
  }
  if (y == nullptr) return;
  sum = block_sum(sum, scratch_one);
  const float scale = rsqrtf(sum / static_cast<float>(size) + eps);
  for (int i = threadIdx.x * 4; i < size; i += blockDim.x * 4) {
    const float4 v = *reinterpret_cast<const float4*>(s_left + i), g = *reinterpret_cast<const float4*>(w + i);
    pair_store4(y + base + i, make_float4(v.x * scale * g.x, v.y * scale * g.y, v.z * scale * g.z, v.w * scale * g.w));
  }
}

}  // namespace mxb

using namespace mxb;

// The widest row both of whose copies fit a block's shared memory beside the small arrays.
MXB_API int mxb_pair_norm_max_size() { return 28000; }

// x: float32 [rows, size], in place; left: [rows, size] of its type, or float32 [left_parts, rows, size]; right:
// [rows, size]; biases float32 [size] or null; wl, wr, w: float32 [size]; y: [rows, size] of y_dtype, or null (then w
// may be null). size a multiple of 4 (8 with a bfloat16 operand), everything 16-byte aligned.
MXB_API int mxb_pair_norm(float* x, const void* left, int left_dtype, int left_parts, const void* right, int right_dtype,
                          const float* left_bias, const float* right_bias, const float* wl, const float* wr,
                          float left_eps, float right_eps, float a, float b, void* y, int y_dtype, const float* w,
                          int rows, int size, float eps, cudaStream_t stream) {
  if (rows <= 0) return 0;
  auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool halves = left_dtype == kBF16 || right_dtype == kBF16 || (y != nullptr && y_dtype == kBF16);
  if (size <= 0 || size > mxb_pair_norm_max_size() || size % (halves ? 8 : 4) != 0 || left_parts < 1 ||
      (left_parts > 1 && left_dtype != kF32) || wl == nullptr || wr == nullptr || (y != nullptr && w == nullptr) ||
      !aligned(x) || !aligned(left) || !aligned(right) || !aligned(left_bias) || !aligned(right_bias) || !aligned(wl) ||
      !aligned(wr) || !aligned(w) || !aligned(y))
    return static_cast<int>(cudaErrorInvalidValue);
  int threads = ((size / 4 + 31) / 32) * 32;
  if (threads > kPairThreads) threads = kPairThreads;
  const int shared = 2 * size * static_cast<int>(sizeof(float));
#define GO(TO)                                                                                                         \
  {                                                                                                                    \
    auto kernel = pair_norm_kernel<TO>;                                                                                \
    if (shared > 40 * 1024) {                                                                                          \
      cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, shared);               \
      if (e != cudaSuccess) return static_cast<int>(e);                                                                \
    }                                                                                                                  \
    return static_cast<int>(launch_chained(kernel, dim3(rows), dim3(threads), shared, stream, x, left, left_dtype,      \
                                           left_parts, right, right_dtype, left_bias, right_bias, wl, wr, left_eps,     \
                                           right_eps, a, b, static_cast<TO*>(y), w, rows, size, eps));                  \
  }
  if (y == nullptr || y_dtype == kF32) GO(float)
  if (y_dtype == kBF16) GO(__nv_bfloat16)
#undef GO
  return static_cast<int>(cudaErrorInvalidValue);
}
