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
// row, four values a thread at a time; both rows wait in registers between the
// passes, or, where they are too wide for that, in shared memory, each value
// read only by the thread that put it there.
#include "common.cuh"

namespace mxb {

constexpr int kPairThreads = 256;

// Four values as loaded, and as floats: the loads of a row are all on their way before the first is looked at.
__device__ __forceinline__ float4 pair_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ uint2 pair_load4(const __nv_bfloat16* p) { return *reinterpret_cast<const uint2*>(p); }
__device__ __forceinline__ float4 pair_floats(float4 raw) { return raw; }
__device__ __forceinline__ float4 pair_floats(uint2 raw) {
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

// Rows of up to 4 * PER * blockDim.x values, held in registers: every load of the row is on its way at once.
template <typename TLeft, typename TRight, typename TOut, int PER>
__global__ void __launch_bounds__(2 * kPairThreads)
pair_norm_held_kernel(float* __restrict__ x, const TLeft* __restrict__ left, int left_parts, const TRight* __restrict__ right,
                      const float* __restrict__ left_bias,
                      const float* __restrict__ right_bias, const float* __restrict__ wl, const float* __restrict__ wr,
                      float left_eps, float right_eps, float a, float b, TOut* __restrict__ y, const float* __restrict__ w,
                      int rows, int size, float eps) {
  __shared__ float2 scratch[2 * kPairThreads / 32];
  __shared__ float scratch_one[33];
  chain_release();
  const size_t base = static_cast<size_t>(blockIdx.x) * size;
  const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  const int step = blockDim.x * 4;
  chain_wait();
  float* row = behind_wait(x) + base;
  left = behind_wait(left);
  right = behind_wait(right);
  float4 l[PER], r[PER], v[PER];
  decltype(pair_load4(left)) raw_left[PER] = {};
  decltype(pair_load4(right)) raw_right[PER] = {};
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int i = threadIdx.x * 4 + p * step;
    v[p] = zero;
    if (i < size) {
      raw_left[p] = pair_load4(left + base + i);
      raw_right[p] = pair_load4(right + base + i);
      v[p] = *reinterpret_cast<const float4*>(row + i);
    }
  }
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    l[p] = pair_floats(raw_left[p]);
    r[p] = pair_floats(raw_right[p]);
  }
  for (int part = 1; part < left_parts; ++part) {
#pragma unroll
    for (int p = 0; p < PER; ++p) {
      const int i = threadIdx.x * 4 + p * step;
      if (i < size) l[p] = pair_sum(l[p], pair_floats(pair_load4(left + static_cast<size_t>(part) * rows * size + base + i)));
    }
  }
  float sum_left = 0.0f, sum_right = 0.0f;
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int i = threadIdx.x * 4 + p * step;
    if (i < size && left_bias != nullptr) l[p] = pair_sum(l[p], *reinterpret_cast<const float4*>(left_bias + i));
    if (i < size && right_bias != nullptr) r[p] = pair_sum(r[p], *reinterpret_cast<const float4*>(right_bias + i));
    sum_left += pair_square(l[p]);
    sum_right += pair_square(r[p]);
  }
  const float2 sums = pair_block_sums(sum_left, sum_right, scratch);
  const float scale_left = a * rsqrtf(sums.x / static_cast<float>(size) + left_eps);
  const float scale_right = b * rsqrtf(sums.y / static_cast<float>(size) + right_eps);
  float sum = 0.0f;
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int i = threadIdx.x * 4 + p * step;
    if (i >= size) continue;
    const float4 gl = *reinterpret_cast<const float4*>(wl + i), gr = *reinterpret_cast<const float4*>(wr + i);
    v[p].x += l[p].x * scale_left * gl.x + r[p].x * scale_right * gr.x;
    v[p].y += l[p].y * scale_left * gl.y + r[p].y * scale_right * gr.y;
    v[p].z += l[p].z * scale_left * gl.z + r[p].z * scale_right * gr.z;
    v[p].w += l[p].w * scale_left * gl.w + r[p].w * scale_right * gr.w;
    *reinterpret_cast<float4*>(row + i) = v[p];
    sum += pair_square(v[p]);
  }
  if (y == nullptr) return;
  sum = block_sum(sum, scratch_one);
  const float scale = rsqrtf(sum / static_cast<float>(size) + eps);
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int i = threadIdx.x * 4 + p * step;
    if (i >= size) continue;
    const float4 g = *reinterpret_cast<const float4*>(w + i);
    pair_store4(y + base + i, make_float4(v[p].x * scale * g.x, v[p].y * scale * g.y, v[p].z * scale * g.z, v[p].w * scale * g.w));
  }
}

// Wider rows wait in shared memory between the passes.
template <typename TLeft, typename TRight, typename TOut>
__global__ void __launch_bounds__(kPairThreads)
pair_norm_kernel(float* __restrict__ x, const TLeft* __restrict__ left, int left_parts, const TRight* __restrict__ right,
                 const float* __restrict__ left_bias,
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
    float4 l = pair_floats(pair_load4(left + base + i));
    for (int part = 1; part < left_parts; ++part)
      l = pair_sum(l, pair_floats(pair_load4(left + static_cast<size_t>(part) * rows * size + base + i)));
    if (left_bias != nullptr) l = pair_sum(l, *reinterpret_cast<const float4*>(left_bias + i));
    float4 r = pair_floats(pair_load4(right + base + i));
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
#define ARGS x, static_cast<const TL*>(left), left_parts, static_cast<const TR*>(right), left_bias, right_bias, wl, wr, left_eps, \
             right_eps, a, b, static_cast<TO*>(y), w, rows, size, eps
#define HELD(PER, THREADS) \
  return static_cast<int>(launch_chained(pair_norm_held_kernel<TL, TR, TO, PER>, dim3(rows), dim3(THREADS), 0, stream, ARGS))
  auto go = [&](auto tl, auto tr, auto to) -> int {
    using TL = decltype(tl);
    using TR = decltype(tr);
    using TO = decltype(to);
    if (size <= 4 * kPairThreads) HELD(1, threads);
    if (size <= 8 * kPairThreads) HELD(2, kPairThreads);
    if (size <= 16 * kPairThreads) HELD(4, kPairThreads);
    if (size <= 32 * kPairThreads) HELD(4, 2 * kPairThreads);
    auto kernel = pair_norm_kernel<TL, TR, TO>;
    if (shared > 40 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, shared);
      if (e != cudaSuccess) return static_cast<int>(e);
    }
    return static_cast<int>(launch_chained(kernel, dim3(rows), dim3(threads), shared, stream, ARGS));
  };
  auto by_right = [&](auto tl) -> int {
    const bool wide_out = y == nullptr || y_dtype == kF32;
    if (right_dtype == kF32) return wide_out ? go(tl, float{}, float{}) : go(tl, float{}, __nv_bfloat16{});
    return wide_out ? go(tl, __nv_bfloat16{}, float{}) : go(tl, __nv_bfloat16{}, __nv_bfloat16{});
  };
  for (int code : {left_dtype, right_dtype, y == nullptr ? static_cast<int>(kF32) : y_dtype})
    if (code != kF32 && code != kBF16) return static_cast<int>(cudaErrorInvalidValue);
  return left_dtype == kF32 ? by_right(float{}) : by_right(__nv_bfloat16{});
#undef HELD
#undef ARGS
}
