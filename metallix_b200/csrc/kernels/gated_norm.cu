// The end of a recurrent mixer whose gate comes ahead of its norm:
//
//   u = x * act(gate),   y = u * rsqrt(mean over the part of u^2 + eps) * w
//
// or (`behind`) follows it, y = x * rsqrt(mean over the part of x^2 + eps) * w * act(gate),
// with the row cut into `parts` equal parts, each over its own root mean
// square, and act silu or the sigmoid. x is float32 (what the recurrence
// read), the gate of its own type (a column range of a wider product will
// do), y of the type the projection behind it takes. One block per (row,
// part); u waits in registers between the passes where vectors divide the part
// and it is not too wide, else in shared memory, each value read only by the
// thread that put it there.
#include "common.cuh"

namespace mxb {

constexpr int kGatedNormThreads = 256;

__device__ __forceinline__ float gate_value(float z, int silu) { return silu ? z * sigmoid_of(z) : sigmoid_of(z); }

template <typename TGate, typename TOut>
__global__ void __launch_bounds__(kGatedNormThreads)
gated_norm_kernel(const float* __restrict__ x, const TGate* __restrict__ gate, long long ldg, const float* __restrict__ w,
                  TOut* __restrict__ y, int parts, int part_size, int silu, int behind, float eps) {
  extern __shared__ float gated_row[];
  __shared__ float scratch[33];
  const int t = blockIdx.x / parts, part = blockIdx.x - t * parts;
  const size_t base = (static_cast<size_t>(t) * parts + part) * part_size;
  const TGate* g = gate + static_cast<long long>(t) * ldg + static_cast<long long>(part) * part_size;
  float sum = 0.0f;
  for (int i = threadIdx.x; i < part_size; i += blockDim.x) {
    const float u = behind ? x[base + i] : x[base + i] * gate_value(to_float(g[i]), silu);
    gated_row[i] = u;
    sum = fmaf(u, u, sum);
  }
  sum = block_sum(sum, scratch);
  const float scale = rsqrtf(sum / static_cast<float>(part_size) + eps);
  const float* weight = w + static_cast<size_t>(part) * part_size;
  for (int i = threadIdx.x; i < part_size; i += blockDim.x)
    y[base + i] = from_float<TOut>(gated_row[i] * scale * weight[i] * (behind ? gate_value(to_float(g[i]), silu) : 1.0f));
}

__device__ __forceinline__ float4 gated_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 gated_load4(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(raw.x << 16), __uint_as_float(raw.x & 0xffff0000u),
                     __uint_as_float(raw.y << 16), __uint_as_float(raw.y & 0xffff0000u));
}
__device__ __forceinline__ void gated_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void gated_store4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
}

// The same for parts of up to 4 * PER * blockDim.x values that vectors divide: the part waits in registers.
template <typename TGate, typename TOut, int PER>
__global__ void __launch_bounds__(2 * kGatedNormThreads)
gated_norm_held_kernel(const float* __restrict__ x, const TGate* __restrict__ gate, long long ldg,
                       const float* __restrict__ w, TOut* __restrict__ y, int parts, int part_size, int silu, int behind, float eps) {
  __shared__ float scratch[33];
  const int t = blockIdx.x / parts, part = blockIdx.x - t * parts;
  const size_t base = (static_cast<size_t>(t) * parts + part) * part_size;
  const TGate* g = gate + static_cast<long long>(t) * ldg + static_cast<long long>(part) * part_size;
  const int step = blockDim.x * 4;
  const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  float4 u[PER], z[PER];
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int i = threadIdx.x * 4 + p * step;
    u[p] = i < part_size ? gated_load4(x + base + i) : zero;
    z[p] = i < part_size ? gated_load4(g + i) : zero;
  }
  float sum = 0.0f;
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    z[p] = make_float4(gate_value(z[p].x, silu), gate_value(z[p].y, silu), gate_value(z[p].z, silu), gate_value(z[p].w, silu));
    if (!behind) { u[p].x *= z[p].x; u[p].y *= z[p].y; u[p].z *= z[p].z; u[p].w *= z[p].w; }
    sum += u[p].x * u[p].x + u[p].y * u[p].y + u[p].z * u[p].z + u[p].w * u[p].w;
  }
  sum = block_sum(sum, scratch);
  const float scale = rsqrtf(sum / static_cast<float>(part_size) + eps);
  const float* weight = w + static_cast<size_t>(part) * part_size;
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int i = threadIdx.x * 4 + p * step;
    if (i >= part_size) continue;
    float4 gain = gated_load4(weight + i);
    if (behind) { gain.x *= z[p].x; gain.y *= z[p].y; gain.z *= z[p].z; gain.w *= z[p].w; }
    gated_store4(y + base + i, make_float4(u[p].x * scale * gain.x, u[p].y * scale * gain.y, u[p].z * scale * gain.z, u[p].w * scale * gain.w));
  }
}

}  // namespace mxb

using namespace mxb;

MXB_API int mxb_gated_norm_max_part() { return 48000; }

// x: float32 [tokens, parts * part_size]; gate: the same shape, rows ldg apart; w: float32 [parts * part_size];
// y: [tokens, parts * part_size]. silu: the gate's activation is silu, else the sigmoid;
// behind: the gate multiplies what the norm leaves, else what it takes.
MXB_API int mxb_gated_norm(const float* x, const void* gate, long long ldg, int gate_dtype, const float* w, void* y,
                           int out_dtype, int tokens, int parts, int part_size, int silu, int behind, float eps, cudaStream_t stream) {
  const long long blocks = static_cast<long long>(tokens) * parts;
  if (blocks <= 0) return 0;
  if (part_size <= 0 || part_size > mxb_gated_norm_max_part() || blocks > 0x7fffffffLL)
    return static_cast<int>(cudaErrorInvalidValue);
  int threads = 32;
  while (threads < part_size && threads < kGatedNormThreads) threads <<= 1;
  const int shared = part_size * static_cast<int>(sizeof(float));
  auto aligned = [](const void* p, int bytes) { return reinterpret_cast<uintptr_t>(p) % bytes == 0; };
  const bool vectors = part_size % 4 == 0 && ldg % 4 == 0 && part_size <= 32 * kGatedNormThreads && aligned(x, 16) &&
                       aligned(w, 16) && aligned(gate, gate_dtype == kF32 ? 16 : 8) && aligned(y, out_dtype == kF32 ? 16 : 8);
  int held = ((part_size / 4 + 31) / 32) * 32;     // threads: a vector each, up to 256; then more vectors, then 512
  if (held > kGatedNormThreads) held = part_size <= 16 * kGatedNormThreads ? kGatedNormThreads : 2 * kGatedNormThreads;
#define LAUNCH(TG, TO)                                                                                                  \
  if (vectors) {                                                                                                        \
    if (part_size <= 4 * held)                                                                                          \
      gated_norm_held_kernel<TG, TO, 1><<<static_cast<unsigned>(blocks), held, 0, stream>>>(                            \
          x, static_cast<const TG*>(gate), ldg, w, static_cast<TO*>(y), parts, part_size, silu, behind, eps);                   \
    else                                                                                                                \
      gated_norm_held_kernel<TG, TO, 4><<<static_cast<unsigned>(blocks), held, 0, stream>>>(                            \
          x, static_cast<const TG*>(gate), ldg, w, static_cast<TO*>(y), parts, part_size, silu, behind, eps);                   \
  } else {                                                                                                              \
    auto kernel = gated_norm_kernel<TG, TO>;                                                                            \
    if (shared > 40 * 1024) {                                                                                           \
      cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, shared);                \
      if (e != cudaSuccess) return static_cast<int>(e);                                                                 \
    }                                                                                                                   \
    kernel<<<static_cast<unsigned>(blocks), threads, shared, stream>>>(x, static_cast<const TG*>(gate), ldg, w,          \
                                                                       static_cast<TO*>(y), parts, part_size, silu, behind, eps); \
  }
  if (gate_dtype == kF32 && out_dtype == kF32) LAUNCH(float, float)
  else if (gate_dtype == kF32 && out_dtype == kBF16) LAUNCH(float, __nv_bfloat16)
  else if (gate_dtype == kBF16 && out_dtype == kF32) LAUNCH(__nv_bfloat16, float)
  else if (gate_dtype == kBF16 && out_dtype == kBF16) LAUNCH(__nv_bfloat16, __nv_bfloat16)
  else return static_cast<int>(cudaErrorInvalidValue);
#undef LAUNCH
  return static_cast<int>(cudaGetLastError());
}
