// The end of a recurrent mixer whose gate comes ahead of its norm:
//
//   u = x * act(gate),   y = u * rsqrt(mean over the part of u^2 + eps) * w
//
// with the row cut into `parts` equal parts, each over its own root mean
// square, and act silu or the sigmoid. x is float32 (what the recurrence
// read), the gate of its own type (a column range of a wider product will
// do), y of the type the projection behind it takes. One block per (row,
// part); u waits in shared memory between the passes, each value read only by
// the thread that put it there.
#include "common.cuh"

namespace mxb {

constexpr int kGatedNormThreads = 256;

template <typename TGate, typename TOut>
__global__ void __launch_bounds__(kGatedNormThreads)
gated_norm_kernel(const float* __restrict__ x, const TGate* __restrict__ gate, long long ldg, const float* __restrict__ w,
                  TOut* __restrict__ y, int parts, int part_size, int silu, float eps) {
  extern __shared__ float gated_row[];
  __shared__ float scratch[33];
  const int t = blockIdx.x / parts, part = blockIdx.x - t * parts;
  const size_t base = (static_cast<size_t>(t) * parts + part) * part_size;
  const TGate* g = gate + static_cast<long long>(t) * ldg + static_cast<long long>(part) * part_size;
  float sum = 0.0f;
  for (int i = threadIdx.x; i < part_size; i += blockDim.x) {
    const float z = to_float(g[i]);
    const float u = x[base + i] * (silu ? z * sigmoid_of(z) : sigmoid_of(z));
    gated_row[i] = u;
    sum = fmaf(u, u, sum);
  }
  sum = block_sum(sum, scratch);
  const float scale = rsqrtf(sum / static_cast<float>(part_size) + eps);
  const float* weight = w + static_cast<size_t>(part) * part_size;
  for (int i = threadIdx.x; i < part_size; i += blockDim.x) y[base + i] = from_float<TOut>(gated_row[i] * scale * weight[i]);
}

}  // namespace mxb

using namespace mxb;

MXB_API int mxb_gated_norm_max_part() { return 48000; }

// x: float32 [tokens, parts * part_size]; gate: the same shape, rows ldg apart; w: float32 [parts * part_size];
// y: [tokens, parts * part_size]. silu: the gate's activation is silu, else the sigmoid.
MXB_API int mxb_gated_norm(const float* x, const void* gate, long long ldg, int gate_dtype, const float* w, void* y,
                           int out_dtype, int tokens, int parts, int part_size, int silu, float eps, cudaStream_t stream) {
  const long long blocks = static_cast<long long>(tokens) * parts;
  if (blocks <= 0) return 0;
  if (part_size <= 0 || part_size > mxb_gated_norm_max_part() || blocks > 0x7fffffffLL)
    return static_cast<int>(cudaErrorInvalidValue);
  int threads = 32;
  while (threads < part_size && threads < kGatedNormThreads) threads <<= 1;
  const int shared = part_size * static_cast<int>(sizeof(float));
#define LAUNCH(TG, TO)                                                                                                  \
  {                                                                                                                     \
    auto kernel = gated_norm_kernel<TG, TO>;                                                                            \
    if (shared > 40 * 1024) {                                                                                           \
      cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, shared);                \
      if (e != cudaSuccess) return static_cast<int>(e);                                                                 \
    }                                                                                                                   \
    kernel<<<static_cast<unsigned>(blocks), threads, shared, stream>>>(x, static_cast<const TG*>(gate), ldg, w,          \
                                                                       static_cast<TO*>(y), parts, part_size, silu, eps); \
  }
  if (gate_dtype == kF32 && out_dtype == kF32) LAUNCH(float, float)
  else if (gate_dtype == kF32 && out_dtype == kBF16) LAUNCH(float, __nv_bfloat16)
  else if (gate_dtype == kBF16 && out_dtype == kF32) LAUNCH(__nv_bfloat16, float)
  else if (gate_dtype == kBF16 && out_dtype == kBF16) LAUNCH(__nv_bfloat16, __nv_bfloat16)
  else return static_cast<int>(cudaErrorInvalidValue);
#undef LAUNCH
  return static_cast<int>(cudaGetLastError());
}
