// Lightning attention: linear attention whose decay per head is a constant.
//
// Over portions of prompts, on the tensor cores in chunks of 64 tokens. Per
// head, with g the decay and q, k, v past their silu (rounded to bfloat16, as
// the token-by-token form in delta_rule.cu rounds them),
//
//   S <- g S + k v^T,   o = S^T q
//
// so that over a chunk of n tokens that begins with state S
//
//   o_i = g^(i+1) S^T q_i + sum_(j <= i) g^(i-j) (q_i . k_j) v_j
//   S  <- g^n S + sum_j g^(n-1-j) k_j v_j^T
//
// A block owns 32 value columns of one head of one request and walks over the
// request's chunks. Warps 0..3 take 16 tokens each: the scores q k^T below the
// diagonal, times their powers of g, times v. Warps 4..7 take the same tokens'
// share of the old state, q S, and then the state itself, of which each keeps
// a quarter of the key channels in float32 registers. Operands of the tensor
// cores are bfloat16: q, k and v are that already; the scores, the state and
// g^(n-1-j) v are float32 numbers, each cut into two bfloat16 parts (the value
// and what its rounding left), whose two products are added up in float32: 16
// bits of each number take part. The state in its registers is never rounded.
//
// silu is applied by a pass of its own ahead of the chunks: several blocks read
// the same queries and keys, and the exponentials of 64 tokens cost a block as
// much time as its products. The next chunk's rows are on their way (cp.async)
// while this one is worked on.
//
// Over single tokens (and a few) the state is what must be read and written:
// lightning_step_kernel gives a value column to 8, 16 or 32 lanes with four key
// channels each, a warp several columns whose loads are all on their way at
// once, and walks over the row's tokens with the state in registers.
#include "common.cuh"

namespace mxb {

constexpr int kLnTokens = 64;       // of a chunk
constexpr int kLnColumns = 32;      // value columns of a block
constexpr int kLnThreads = 256;
constexpr int kLnValuePitch = kLnColumns * 2 + 16;   // bytes of a row of values: eight rows fall on eight bank groups
constexpr int kLnSumPitch = kLnColumns + 4;          // floats of a row of the old state's share

template <int DP> struct LnLayout {                  // DP: key channels, padded with zeros to 64 or 128
  static constexpr int kPitch = DP * 2 + 16;         // bytes of a row of queries or keys
  static constexpr int kRows = kLnTokens * kPitch;   // q or k of a chunk
  static constexpr int kValues = kLnTokens * kLnValuePitch;
  static constexpr int kStage = 2 * kRows + 3 * kValues;          // q, k, v, and g^(n-1-j) v in two parts
  static constexpr int kState = DP * kLnValuePitch;               // one part of the state
  static constexpr int kSums = kLnTokens * kLnSumPitch * 4;
  static constexpr int kPowers = (kLnTokens + 4) * 4;
  static constexpr int kBytes = 2 * kStage + 2 * kState + kSums + kPowers;
};

__device__ __forceinline__ uint32_t ln_address(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void ln_copy16(uint32_t dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(live ? 16 : 0));
}
__device__ __forceinline__ void ln_load4(uint32_t (&r)[4], uint32_t address) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(address) : "memory");
}
__device__ __forceinline__ void ln_load4_trans(uint32_t (&r)[4], uint32_t address) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(address) : "memory");
}
__device__ __forceinline__ void ln_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};\n"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two float32 numbers as their bfloat16 values (`high`) and what that rounding left, as bfloat16 too.
__device__ __forceinline__ void ln_split(float x, float y, uint32_t& high, uint32_t& rest) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 back = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - back.x, y - back.y);
  high = *reinterpret_cast<const uint32_t*>(&h);
  rest = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float ln_silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
__device__ __forceinline__ uint32_t ln_silu2(uint32_t pair) {
  const __nv_bfloat162 out = __floats2bfloat162_rn(ln_silu(__uint_as_float(pair << 16)), ln_silu(__uint_as_float(pair & 0xffff0000u)));
  return *reinterpret_cast<const uint32_t*>(&out);
}

// x[t, c] <- silu(x[t, c]) rounded, for eight neighbouring columns a thread: a column range of a wider matrix, in place.
__global__ void __launch_bounds__(256)
silu_columns_kernel(__nv_bfloat16* __restrict__ x, long long ld, int pieces, long long total) {
  const long long index = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (index >= total) return;
  const long long token = index / pieces;
  uint4* p = reinterpret_cast<uint4*>(x + token * ld + (index - token * pieces) * 8);
  uint4 raw = *p;
  raw.x = ln_silu2(raw.x); raw.y = ln_silu2(raw.y); raw.z = ln_silu2(raw.z); raw.w = ln_silu2(raw.w);
  *p = raw;
}

__device__ __forceinline__ void ln_meet(int id, int threads) { asm volatile("bar.sync %0, %1;\n" ::"r"(id), "r"(threads) : "memory"); }
__device__ __forceinline__ void ln_arrive(int id, int threads) { asm volatile("bar.arrive %0, %1;\n" ::"r"(id), "r"(threads) : "memory"); }

template <int DP>
__global__ void __launch_bounds__(kLnThreads)
lightning_chunk_kernel(const __nv_bfloat16* __restrict__ qkv, long long ld, int q_off, int k_off, int v_off,
                       const float* __restrict__ decay, float* __restrict__ state, long long slot_stride, int num_slots,
                       const int* __restrict__ row_start, const int* __restrict__ row_length,
                       const int* __restrict__ request_slots, float* __restrict__ out, int heads, int dim, int vdim,
                       int* status) {
  using Layout = LnLayout<DP>;
  constexpr int PITCH = Layout::kPitch;
  constexpr int TILES = DP / 64;              // 16-row tiles of the state that a warp keeps: a quarter of the channels
  constexpr int PIECES = DP / 8;              // 16-byte pieces of a row of queries or keys
  extern __shared__ __align__(128) unsigned char ln_shared[];
  const int row = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * kLnColumns;
  const int length = row_length[row];
  if (length <= 0) return;   // a padding row owns no state
  const int slot = request_slots[row];
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0) atomicOr(status, kStatusBadSlot);
    return;
  }
  const int first = row_start[row];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = lane >> 2, t = lane & 3;
  unsigned char* s_state = ln_shared + 2 * Layout::kStage;        // its bfloat16 values, then what they leave
  float* s_sums = reinterpret_cast<float*>(s_state + 2 * Layout::kState);
  float* s_power = s_sums + kLnTokens * kLnSumPitch;              // g^0 .. g^64
  const float head_decay = decay[head];
  if (tid <= kLnTokens) s_power[tid] = powf(head_decay, static_cast<float>(tid));

  // ---- copies: q and k rows of DP channels (those beyond dim are zeros), 32 value columns, rows beyond the end zeros
  auto fetch = [&](int base, int stage) {
    unsigned char* buffer = ln_shared + stage * Layout::kStage;
    const int live_rows = min(kLnTokens, length - base);
    for (int i = tid; i < 2 * kLnTokens * PIECES; i += kLnThreads) {
      const int which = i / (kLnTokens * PIECES), at = i - which * (kLnTokens * PIECES);
      const int token = at / PIECES, piece = at - token * PIECES;
      const bool live = token < live_rows && piece * 8 < dim;
      const __nv_bfloat16* src = qkv + static_cast<long long>(first + base + (live ? token : 0)) * ld +
                                 (which ? k_off : q_off) + head * dim + (live ? piece * 8 : 0);
      ln_copy16(ln_address(buffer + which * Layout::kRows + token * PITCH + piece * 16), src, live);
    }
    {   // 64 rows of 4 pieces: one a thread
      const int token = tid >> 2, piece = tid & 3;
      const bool live = token < live_rows && v0 + piece * 8 < vdim;
      const __nv_bfloat16* src = qkv + static_cast<long long>(first + base + (live ? token : 0)) * ld + v_off +
                                 head * vdim + (live ? v0 + piece * 8 : 0);
      ln_copy16(ln_address(buffer + 2 * Layout::kRows + token * kLnValuePitch + piece * 16), src, live);
    }
    asm volatile("cp.async.commit_group;\n" ::);
  };
  // ---- the values this thread copied times g^(n-1-j), in two parts
  auto weigh = [&](int base, int stage) {
    unsigned char* buffer = ln_shared + stage * Layout::kStage;
    const int live_rows = min(kLnTokens, length - base);
    const int token = tid >> 2, piece = tid & 3;
    unsigned char* p = buffer + 2 * Layout::kRows + token * kLnValuePitch + piece * 16;
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const float power = token < live_rows ? s_power[live_rows - 1 - token] : 0.0f;
    const uint32_t words[4] = {raw.x, raw.y, raw.z, raw.w};
    uint32_t high[4], rest[4];
#pragma unroll
    for (int w = 0; w < 4; ++w)
      ln_split(__uint_as_float(words[w] << 16) * power, __uint_as_float(words[w] & 0xffff0000u) * power, high[w], rest[w]);
    *reinterpret_cast<uint4*>(p + Layout::kValues) = make_uint4(high[0], high[1], high[2], high[3]);
    *reinterpret_cast<uint4*>(p + 2 * Layout::kValues) = make_uint4(rest[0], rest[1], rest[2], rest[3]);
  };

  // ---- the state: warps 4..7, accumulator fragments of 16-row tiles (key channels) by 8 columns
  float s[TILES][4][4];
  const int keeper = warp - 4;
  auto state_at = [&](int tile, int nb, int e, int& channel, int& column) {
    channel = (keeper * TILES + tile) * 16 + g + (e >> 1) * 8;
    column = v0 + nb * 8 + 2 * t + (e & 1);
    return state + static_cast<long long>(slot) * slot_stride +
           (static_cast<long long>(head) * vdim + column) * dim + channel;
  };
  auto publish = [&]() {   // the state's two parts for the next chunk's products
#pragma unroll
    for (int tile = 0; tile < TILES; ++tile)
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t high, rest;
          ln_split(s[tile][nb][2 * half], s[tile][nb][2 * half + 1], high, rest);
          const int channel = (keeper * TILES + tile) * 16 + g + half * 8;
          unsigned char* p = s_state + channel * kLnValuePitch + (nb * 8 + 2 * t) * 2;
          *reinterpret_cast<uint32_t*>(p) = high;
          *reinterpret_cast<uint32_t*>(p + Layout::kState) = rest;
        }
  };
  fetch(0, 0);
  if (warp >= 4) {
#pragma unroll
    for (int tile = 0; tile < TILES; ++tile)
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          int channel, column;
          const float* p = state_at(tile, nb, e, channel, column);
          s[tile][nb][e] = channel < dim && column < vdim ? *p : 0.0f;
        }
    publish();
  }
  __syncthreads();   // the powers

  int stage = 0;
  for (int base = 0; base < length; base += kLnTokens, stage ^= 1) {
    const int live_rows = min(kLnTokens, length - base);
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    weigh(base, stage);
    __syncthreads();   // this chunk's rows are ready, and the other stage has been read
    if (base + kLnTokens < length) fetch(base + kLnTokens, stage ^ 1);
    const unsigned char* s_q = ln_shared + stage * Layout::kStage;
    const unsigned char* s_k = s_q + Layout::kRows;
    const unsigned char* s_v = s_k + Layout::kRows;
    // this warp's 16 tokens as the row operand: row (lane & 15), 8 channels further for the upper half of the lanes
    const int token0 = (warp & 3) * 16;
    const uint32_t q_frag = ln_address(s_q + (token0 + (lane & 15)) * PITCH + (lane >> 4) * 16);
    // 16 rows (tokens or channels) of 16 columns, transposed: the column operand of a product over those rows
    const int across = (lane & 15) * kLnValuePitch + (lane >> 4) * 16;

    if (warp < 4) {
      // ---- scores below the diagonal: keys in runs of 16, as many as reach this warp's tokens
      float o[4][4];
#pragma unroll
      for (int nb = 0; nb < 4; ++nb) o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.0f;
      if (token0 < live_rows) {
        uint32_t q[DP / 16][4];
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks) ln_load4(q[ks], q_frag + ks * 32);
        for (int run = 0; run <= (warp & 3); ++run) {
          float p[2][4];
          p[0][0] = p[0][1] = p[0][2] = p[0][3] = p[1][0] = p[1][1] = p[1][2] = p[1][3] = 0.0f;
          const uint32_t k_frag = ln_address(s_k + (run * 16 + (lane & 7) + (lane >> 4) * 8) * PITCH + ((lane >> 3) & 1) * 16);
#pragma unroll
          for (int ks = 0; ks < DP / 16; ++ks) {
            uint32_t k[4];
            ln_load4(k, k_frag + ks * 32);
            ln_mma(p[0], q[ks], k[0], k[1]);
            ln_mma(p[1], q[ks], k[2], k[3]);
          }
          // token i = token0 + g (+ 8), key j = 16 run + 8 n + 2 t (+ 1): times g^(i-j), nothing above the diagonal
          uint32_t high[4], rest[4];
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const int back = token0 + g - (run * 16 + n * 8 + 2 * t);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int distance = back + (e >> 1) * 8 - (e & 1);
              p[n][e] = distance >= 0 ? p[n][e] * s_power[distance] : 0.0f;
            }
            ln_split(p[n][0], p[n][1], high[2 * n], rest[2 * n]);
            ln_split(p[n][2], p[n][3], high[2 * n + 1], rest[2 * n + 1]);
          }
          const uint32_t v_frag = ln_address(s_v + run * 16 * kLnValuePitch + across);
#pragma unroll
          for (int pair = 0; pair < 2; ++pair) {
            uint32_t v[4];
            ln_load4_trans(v, v_frag + pair * 32);
            ln_mma(o[2 * pair], high, v[0], v[1]);
            ln_mma(o[2 * pair + 1], high, v[2], v[3]);
            ln_mma(o[2 * pair], rest, v[0], v[1]);
            ln_mma(o[2 * pair + 1], rest, v[2], v[3]);
          }
        }
      }
      ln_meet(2, kLnThreads);   // the old state's share has been left in s_sums
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int token = token0 + g + half * 8;
        if (token >= live_rows) continue;
        float* dst = out + static_cast<long long>(first + base + token) * (static_cast<long long>(heads) * vdim) + head * vdim + v0;
        const float* old = s_sums + token * kLnSumPitch;
#pragma unroll
        for (int nb = 0; nb < 4; ++nb) {
          const int column = nb * 8 + 2 * t;     // vdim is a multiple of 8: a pair of columns is there or not
          if (v0 + column >= vdim) continue;
          const float2 before = *reinterpret_cast<const float2*>(old + column);
          *reinterpret_cast<float2*>(dst + column) = make_float2(o[nb][2 * half] + before.x, o[nb][2 * half + 1] + before.y);
        }
      }
    } else {
      // ---- the old state's share of these tokens, g^(i+1) S^T q_i
      float o[4][4];
#pragma unroll
      for (int nb = 0; nb < 4; ++nb) o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.0f;
      if (token0 < live_rows) {
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks) {
          uint32_t q[4];
          ln_load4(q, q_frag + ks * 32);
          const uint32_t s_frag = ln_address(s_state + ks * 16 * kLnValuePitch + across);
#pragma unroll
          for (int pair = 0; pair < 2; ++pair) {
            uint32_t high[4], rest[4];
            ln_load4_trans(high, s_frag + pair * 32);
            ln_load4_trans(rest, s_frag + Layout::kState + pair * 32);
            ln_mma(o[2 * pair], q, high[0], high[1]);
            ln_mma(o[2 * pair + 1], q, high[2], high[3]);
            ln_mma(o[2 * pair], q, rest[0], rest[1]);
            ln_mma(o[2 * pair + 1], q, rest[2], rest[3]);
          }
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int token = token0 + g + half * 8;
          const float power = s_power[token + 1];
#pragma unroll
          for (int nb = 0; nb < 4; ++nb)
            *reinterpret_cast<float2*>(s_sums + token * kLnSumPitch + nb * 8 + 2 * t) =
                make_float2(o[nb][2 * half] * power, o[nb][2 * half + 1] * power);
        }
      }
      ln_arrive(2, kLnThreads);
      ln_meet(1, 128);           // every keeper has read the old state's two parts
      // ---- the new state: this warp's channels by the block's columns, over the chunk's tokens
      const float fade = s_power[live_rows];
#pragma unroll
      for (int tile = 0; tile < TILES; ++tile)
#pragma unroll
        for (int nb = 0; nb < 4; ++nb)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[tile][nb][e] *= fade;
      for (int run = 0; run * 16 < live_rows; ++run) {
        uint32_t high[2][4], rest[2][4];
        const uint32_t v_frag = ln_address(s_v + Layout::kValues + run * 16 * kLnValuePitch + across);
#pragma unroll
        for (int pair = 0; pair < 2; ++pair) {
          ln_load4_trans(high[pair], v_frag + pair * 32);
          ln_load4_trans(rest[pair], v_frag + Layout::kValues + pair * 32);
        }
#pragma unroll
        for (int tile = 0; tile < TILES; ++tile) {
          // keys transposed: 16 channels as rows, 16 tokens as columns
          uint32_t k[4];
          ln_load4_trans(k, ln_address(s_k + (run * 16 + (lane & 7) + (lane >> 4) * 8) * PITCH +
                                       ((keeper * TILES + tile) * 16 + ((lane >> 3) & 1) * 8) * 2));
#pragma unroll
          for (int pair = 0; pair < 2; ++pair) {
            ln_mma(s[tile][2 * pair], k, high[pair][0], high[pair][1]);
            ln_mma(s[tile][2 * pair + 1], k, high[pair][2], high[pair][3]);
            ln_mma(s[tile][2 * pair], k, rest[pair][0], rest[pair][1]);
            ln_mma(s[tile][2 * pair + 1], k, rest[pair][2], rest[pair][3]);
          }
        }
      }
      publish();
    }
  }
  if (warp >= 4) {
#pragma unroll
    for (int tile = 0; tile < TILES; ++tile)
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          int channel, column;
          float* p = state_at(tile, nb, e, channel, column);
          if (channel < dim && column < vdim) *p = s[tile][nb][e];
        }
  }
}

// Four neighbouring values as floats past their silu, rounded to their own type.
__device__ __forceinline__ float4 ln_silu_four(const float* p) {
  const float4 x = *reinterpret_cast<const float4*>(p);
  return make_float4(x.x * sigmoid_of(x.x), x.y * sigmoid_of(x.y), x.z * sigmoid_of(x.z), x.w * sigmoid_of(x.w));
}
__device__ __forceinline__ float ln_silu_half(uint32_t bits) {
  const float z = __uint_as_float(bits);
  return to_float(from_float<__nv_bfloat16>(z * sigmoid_of(z)));
}
__device__ __forceinline__ float4 ln_silu_four(const __nv_bfloat16* p) {
  const uint2 x = *reinterpret_cast<const uint2*>(p);
  return make_float4(ln_silu_half(x.x << 16), ln_silu_half(x.x & 0xffff0000u), ln_silu_half(x.y << 16),
                     ln_silu_half(x.y & 0xffff0000u));
}

// LANES lanes share a column (four of its key channels each), so a warp holds 32 / LANES columns side by side, kLnHeld of
// each lane; a block is kLnStepWarps warps.
constexpr int kLnHeld = 4, kLnStepWarps = 4;

template <typename T, int LANES>
__global__ void __launch_bounds__(kLnStepWarps * 32)
lightning_step_kernel(const T* __restrict__ qkv, long long ld, int q_off, int k_off, int v_off,
                      const float* __restrict__ decay, float* __restrict__ state, long long slot_stride, int num_slots,
                      const int* __restrict__ row_start, const int* __restrict__ row_length,
                      const int* __restrict__ request_slots, float* __restrict__ out, int heads, int dim, int vdim,
                      int* status) {
  constexpr int SIDE = 32 / LANES, COLUMNS = SIDE * kLnHeld;     // columns of a warp
  const int row = blockIdx.x, head = blockIdx.y;
  const int length = row_length[row], slot = request_slots[row], first = row_start[row];
  if (length <= 0) return;   // a padding row owns no state
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0) atomicOr(status, kStatusBadSlot);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, side = lane / LANES, d = (lane % LANES) * 4;
  const int column0 = (blockIdx.z * kLnStepWarps + warp) * COLUMNS + side;   // this lane's columns: column0 + c * SIDE
  const bool channels = d < dim;
  float* base = state + static_cast<long long>(slot) * slot_stride + static_cast<long long>(head) * vdim * dim + d;
  float4 s[kLnHeld];
#pragma unroll
  for (int c = 0; c < kLnHeld; ++c) {
    const int column = column0 + c * SIDE;
    s[c] = channels && column < vdim ? *reinterpret_cast<const float4*>(base + static_cast<long long>(column) * dim)
                                     : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  const float g = decay[head];
  for (int t = 0; t < length; ++t) {
    const T* token = qkv + static_cast<long long>(first + t) * ld;
    float4 q = make_float4(0.0f, 0.0f, 0.0f, 0.0f), k = q;
    if (channels) {
      q = ln_silu_four(token + q_off + head * dim + d);
      k = ln_silu_four(token + k_off + head * dim + d);
    }
    float sums[kLnHeld];
#pragma unroll
    for (int c = 0; c < kLnHeld; ++c) {
      const int column = column0 + c * SIDE;
      float v = 0.0f;
      if (column < vdim) {
        v = to_float(token[v_off + head * vdim + column]);
        v = to_float(from_float<T>(v * sigmoid_of(v)));
      }
      s[c].x = fmaf(k.x, v, g * s[c].x); s[c].y = fmaf(k.y, v, g * s[c].y);
      s[c].z = fmaf(k.z, v, g * s[c].z); s[c].w = fmaf(k.w, v, g * s[c].w);
      sums[c] = fmaf(q.x, s[c].x, fmaf(q.y, s[c].y, fmaf(q.z, s[c].z, q.w * s[c].w)));
    }
    // kLnHeld sums over LANES lanes: every exchange halves the sums a lane still adds up, then the lanes
    static_assert(kLnHeld == 4, "the exchanges below are for four sums");
    const bool upper = (lane & (LANES / 2)) != 0, odd = (lane & (LANES / 4)) != 0;
    float a = upper ? sums[2] : sums[0], b = upper ? sums[3] : sums[1];
    a += __shfl_xor_sync(0xffffffffu, upper ? sums[0] : sums[2], LANES / 2);
    b += __shfl_xor_sync(0xffffffffu, upper ? sums[1] : sums[3], LANES / 2);
    float sum = odd ? b : a;
    sum += __shfl_xor_sync(0xffffffffu, odd ? a : b, LANES / 4);
#pragma unroll
    for (int offset = LANES / 8; offset > 0; offset >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, offset);
    const int column = column0 + ((upper ? 2 : 0) + (odd ? 1 : 0)) * SIDE;
    if (lane % (LANES / 4) == 0 && column < vdim)
      out[static_cast<long long>(first + t) * (static_cast<long long>(heads) * vdim) + head * vdim + column] = sum;
  }
#pragma unroll
  for (int c = 0; c < kLnHeld; ++c) {
    const int column = column0 + c * SIDE;
    if (channels && column < vdim) *reinterpret_cast<float4*>(base + static_cast<long long>(column) * dim) = s[c];
  }
}

}  // namespace mxb

using namespace mxb;

// Whether the form for few tokens takes this layout: up to 128 key channels in whole groups of four, rows and state on
// boundaries that four values make.
MXB_API int mxb_lightning_steps_supported(const void* qkv, long long ld, int q_off, int k_off, const float* state,
                                          long long slot_stride, int dim, int dtype) {
  const int four = dtype == kBF16 ? 8 : 16;
  return (dtype == kBF16 || dtype == kF32) && dim > 0 && dim <= 128 && dim % 4 == 0 && ld % 4 == 0 && q_off % 4 == 0 &&
                 k_off % 4 == 0 && reinterpret_cast<uintptr_t>(qkv) % four == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0 &&
                 slot_stride % 4 == 0 ? 1 : 0;
}

// Operands as for mxb_lightning_chunks, of either type, q, k and v ahead of their silu.
MXB_API int mxb_lightning_steps(const void* qkv, long long ld, int q_off, int k_off, int v_off, const float* decay,
                                float* state, long long slot_stride, int num_slots, const int* row_start,
                                const int* row_length, const int* request_slots, float* out, int rows, int heads, int dim,
                                int vdim, int dtype, int* status, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (heads <= 0 || vdim <= 0 || !mxb_lightning_steps_supported(qkv, ld, q_off, k_off, state, slot_stride, dim, dtype))
    return static_cast<int>(cudaErrorInvalidValue);
  const int lanes = dim <= 32 ? 8 : (dim <= 64 ? 16 : 32);
  const dim3 grid(rows, heads, ceil_div(vdim, kLnStepWarps * kLnHeld * (32 / lanes))), block(kLnStepWarps * 32);
#define GO(T, LANES)                                                                                                    \
  lightning_step_kernel<T, LANES><<<grid, block, 0, stream>>>(static_cast<const T*>(qkv), ld, q_off, k_off, v_off, decay, \
                                                              state, slot_stride, num_slots, row_start, row_length,     \
                                                              request_slots, out, heads, dim, vdim, status)
  if (dtype == kBF16) {
    if (lanes == 8) GO(__nv_bfloat16, 8);
    else if (lanes == 16) GO(__nv_bfloat16, 16);
    else GO(__nv_bfloat16, 32);
  } else {
    if (lanes == 8) GO(float, 8);
    else if (lanes == 16) GO(float, 16);
    else GO(float, 32);
  }
#undef GO
  return static_cast<int>(cudaGetLastError());
}

// Whether the chunked form takes this layout: bfloat16 rows whose heads are whole 16-byte pieces, up to 128 key channels.
MXB_API int mxb_lightning_chunks_supported(const void* qkv, long long ld, int q_off, int k_off, int v_off, int dim, int vdim,
                                           int dtype) {
  return dtype == kBF16 && dim > 0 && dim <= 128 && dim % 8 == 0 && vdim > 0 && vdim % 8 == 0 && ld % 8 == 0 &&
                 q_off % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0 && (reinterpret_cast<uintptr_t>(qkv) & 15) == 0 ? 1 : 0;
}

// x: bfloat16 [tokens, width], rows ld apart, in place; width and ld multiples of 8, 16-byte aligned.
MXB_API int mxb_silu_columns(void* x, long long ld, int tokens, int width, cudaStream_t stream) {
  const long long total = static_cast<long long>(tokens) * (width / 8);
  if (total <= 0) return 0;
  if (width % 8 != 0 || ld % 8 != 0 || ld < width || (reinterpret_cast<uintptr_t>(x) & 15))
    return static_cast<int>(cudaErrorInvalidValue);
  silu_columns_kernel<<<static_cast<unsigned>((total + 255) / 256), 256, 0, stream>>>(static_cast<__nv_bfloat16*>(x), ld,
                                                                                      width / 8, total);
  return static_cast<int>(cudaGetLastError());
}

// qkv: bfloat16 [tokens, ld], holding from the column offsets on heads * dim queries, as many keys and heads * vdim
// values, all past their silu. decay: float32 [heads]. state: float32 [num_slots, heads, vdim, dim], rows slot_stride
// values apart, advanced in place; rows and slots as for the token-by-token form. out: float32 [tokens, heads * vdim].
MXB_API int mxb_lightning_chunks(const void* qkv, long long ld, int q_off, int k_off, int v_off, const float* decay,
                                 float* state, long long slot_stride, int num_slots, const int* row_start,
                                 const int* row_length, const int* request_slots, float* out, int rows, int heads, int dim,
                                 int vdim, int dtype, int* status, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (heads <= 0 || !mxb_lightning_chunks_supported(qkv, ld, q_off, k_off, v_off, dim, vdim, dtype))
    return static_cast<int>(cudaErrorInvalidValue);
  const dim3 grid(rows, heads, (vdim + kLnColumns - 1) / kLnColumns);
  auto go = [&](auto kernel, int shared) -> int {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, shared);
    if (e != cudaSuccess) return static_cast<int>(e);
    kernel<<<grid, kLnThreads, shared, stream>>>(static_cast<const __nv_bfloat16*>(qkv), ld, q_off, k_off, v_off, decay, state,
                                                 slot_stride, num_slots, row_start, row_length, request_slots, out, heads, dim,
                                                 vdim, status);
    return static_cast<int>(cudaGetLastError());
  };
  return dim <= 64 ? go(lightning_chunk_kernel<64>, LnLayout<64>::kBytes) : go(lightning_chunk_kernel<128>, LnLayout<128>::kBytes);
}
