// What stands between one product that holds [q heads | k heads | v heads] of every token and attention over pages, for
// mixers that send each channel of q, k and v through a short causal convolution over time first:
//
//   u     = product + bias                                     (a bias per channel, or none)
//   y_t   = sum_j w[c, j] u_(t - taps + 1 + j)                 over the sequence's own earlier tokens; the inputs before
//                                                              the step's first token come from the request's state slot,
//                                                              which holds zeros at a sequence's start
//   q, k <- the first rotary_dims dims of every head turned by the token's position (either pair layout)
//   q goes to q_out, k and v to the token's cache slot.
//
// A block takes a run of up to kRun tokens and some of their heads, a warp a head at a time: a lane holds the taps of a
// pair of channels in registers and walks the run's tokens with the last taps - 1 inputs beside them, so that every
// input is read once; cos and sin of the run's positions are worked out once per block.  (Prompts, where pairs of channels
// start on boundaries of their size: two neighbouring channels per access, all inputs of a run loaded ahead.)  Where every sequence of the
// step has one token (decoding) a thread also stores its channel's last taps - 1 inputs into the state slot; otherwise
// conv_tail does that afterwards.
//
// Elementwise gates on attention's output (gate_columns): out = in * sigmoid(gate columns of the product) * factor.
#include "common.cuh"
#include "launchers.h"

namespace akv {

namespace {

constexpr int kRun = 8;
constexpr int kConvWarps = 8;

// one channel's walk: the last TAPS - 1 inputs, oldest first
template <int TAPS>
struct Channel {
  float w[TAPS];
  float past[TAPS > 1 ? TAPS - 1 : 1];
  float bias;
};

struct TokenInfo {
  int64_t first;       // row of the sequence's first token in the step
  int offset;          // tokens of the sequence before this one in the step
  int slot;            // state slot, negative: none
  int fresh;           // 1: the inputs before this token are not those the walk holds (the run's or a sequence's first)
};

template <typename T, int TAPS>
__device__ __forceinline__ void channel_start(const ConvPrepParams& p, Channel<TAPS>& ch, int c) {
#pragma unroll
  for (int j = 0; j < TAPS; ++j) ch.w[j] = TAPS <= 4 || j < p.taps ? p.conv[(int64_t)c * p.taps + j] : 0.f;
  ch.bias = p.bias != nullptr ? p.bias[c] : 0.f;
#pragma unroll
  for (int j = 0; j + 1 < TAPS; ++j) ch.past[j] = 0.f;
}

// the convolution's output for channel c of `token`
template <typename T, int TAPS>
__device__ __forceinline__ float channel_step(const ConvPrepParams& p, Channel<TAPS>& ch, const TokenInfo& info,
                                              int64_t token, int c) {
  const T* x = (const T*)p.x + c;
  const int keep = TAPS <= 4 ? TAPS - 1 : p.taps - 1;
  if (info.fresh && keep > 0) {
    const float* before = p.state + (int64_t)(info.slot < 0 ? 0 : info.slot) * p.state_stride + p.tail_off + c;
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j) {
      if (j < keep) {
        const int back = info.offset - keep + j;         // index within the step's tokens of this sequence
        float u = 0.f;
        if (back >= 0) u = to_float<T>(x[(info.first + back) * p.x_stride]) + ch.bias;
        else if (info.slot >= 0) u = before[(int64_t)(keep + back) * p.channels];
        ch.past[j] = u;
      }
    }
  }
  const float u = to_float<T>(x[token * p.x_stride]) + ch.bias;
  float y = 0.f;
#pragma unroll
  for (int j = 0; j + 1 < TAPS; ++j)
    if (j < keep) y = fmaf(ch.w[j], ch.past[j], y);
  float last = ch.w[0];
#pragma unroll
  for (int j = 1; j < TAPS; ++j)
    if (j == keep) last = ch.w[j];
  y = fmaf(last, u, y);
#pragma unroll
  for (int j = 0; j + 1 < TAPS; ++j) {
    if (j + 1 < keep) ch.past[j] = ch.past[j + 1 < TAPS - 1 ? j + 1 : j];
    else if (j + 1 == keep) ch.past[j] = u;
  }
  if (p.keep_tail && info.slot >= 0) {
    float* before = p.state + (int64_t)info.slot * p.state_stride + p.tail_off + c;
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j)
      if (j < keep) before[(int64_t)j * p.channels] = ch.past[j];
  }
  return y;
}

// What a block knows of its run of tokens: where each stands in its sequence, the cache row of each token's first kv head
// (or -1: not stored), and cos and sin of its positions.
__device__ __forceinline__ void run_prologue(const ConvPrepParams& p, int64_t token0, int run, TokenInfo* infos,
                                             int64_t* cache_rows, float2* turn) {
  const int half = p.rotary_dims / 2;
  if (threadIdx.x < run) {
    const int64_t token = token0 + threadIdx.x;
    int lo = 0, hi = p.num_seqs;                             // cu_q[lo] <= token < cu_q[hi]
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (p.cu_q[mid] <= token) lo = mid; else hi = mid;
    }
    TokenInfo info;
    info.first = p.cu_q[lo];
    info.offset = (int)(token - info.first);
    const int slot = p.state_slots[lo];
    info.slot = slot < p.num_slots ? slot : -1;
    info.fresh = threadIdx.x == 0 || info.offset == 0;
    infos[threadIdx.x] = info;
    const int at = p.slots != nullptr ? p.slots[token] : -1;
    int64_t row = -1;
    if (at >= 0) {
      const int page = at / p.page_size;
      if (page >= p.num_pages) set_status(p.status, kBadSlot);
      else row = (int64_t)page * p.num_kv_heads * p.page_size + at % p.page_size;
    }
    cache_rows[threadIdx.x] = row;
  }
  for (int i = threadIdx.x; i < run * half; i += blockDim.x) {
    const int t = i / half, pair = i - t * half;
    float s, c;
    sincosf((float)p.positions[token0 + t] * p.freq[pair], &s, &c);
    turn[i] = make_float2(c * p.factor, s * p.factor);
  }
  __syncthreads();
}

template <typename T, int TAPS>
__global__ void __launch_bounds__(kConvWarps * 32) conv_rotary_prep_kernel(ConvPrepParams p) {
  extern __shared__ __align__(16) float2 turn[];             // [kRun][half]: cos and sin (times the factor)
  __shared__ TokenInfo infos[kRun];
  __shared__ int64_t cache_rows[kRun];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int NH = p.num_heads, NKV = p.num_kv_heads, D = p.head_dim, DV = p.v_dim, half = p.rotary_dims / 2;
  const int64_t token0 = (int64_t)blockIdx.x * p.run;
  const int run = (int)(p.num_tokens - token0 < p.run ? p.num_tokens - token0 : p.run);
  run_prologue(p, token0, run, infos, cache_rows, turn);
  for (int h = blockIdx.y * kConvWarps + warp; h < NH + 2 * NKV; h += gridDim.y * kConvWarps) {
    const bool is_q = h < NH, is_v = h >= NH + NKV;
    const int g = is_q ? h : (is_v ? h - NH - NKV : h - NH);
    const int width = is_v ? DV : D;
    const int first = is_q ? g * D : (is_v ? (NH + NKV) * D + g * DV : NH * D + g * D);
    auto row_of = [&](int t) -> T* {
      if (is_q) return (T*)p.q_out + ((token0 + t) * NH + g) * (int64_t)D;
      if (cache_rows[t] < 0) return nullptr;
      const int64_t row = cache_rows[t] + (int64_t)g * p.page_size;
      return is_v ? (T*)p.v_cache + row * p.v_row_stride : (T*)p.k_cache + row * p.k_row_stride;
    };
    const int turned = is_v ? 0 : half;
    for (int i = lane; i < turned; i += 32) {
      const int a = p.layout == 0 ? i : 2 * i, b = p.layout == 0 ? i + half : 2 * i + 1;
      Channel<TAPS> ca, cb;
      channel_start<T, TAPS>(p, ca, first + a);
      channel_start<T, TAPS>(p, cb, first + b);
      for (int t = 0; t < run; ++t) {
        const float u = channel_step<T, TAPS>(p, ca, infos[t], token0 + t, first + a);
        const float v = channel_step<T, TAPS>(p, cb, infos[t], token0 + t, first + b);
        const float2 cs = turn[t * half + i];
        T* dst = row_of(t);
        if (dst != nullptr) {
          dst[a] = from_float<T>(u * cs.x - v * cs.y);
          dst[b] = from_float<T>(v * cs.x + u * cs.y);
        }
      }
    }
    for (int d = 2 * turned + lane; d < width; d += 32) {
      Channel<TAPS> ch;
      channel_start<T, TAPS>(p, ch, first + d);
      for (int t = 0; t < run; ++t) {
        const float y = channel_step<T, TAPS>(p, ch, infos[t], token0 + t, first + d);
        T* dst = row_of(t);
        if (dst != nullptr) dst[d] = from_float<T>(y);
      }
    }
  }
}

// Two neighbouring elements in one access
template <typename T>
__device__ __forceinline__ float2 load2(const T* p);
template <>
__device__ __forceinline__ float2 load2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <>
__device__ __forceinline__ float2 load2<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint32_t raw = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(__uint_as_float(raw << 16), __uint_as_float(raw & 0xffff0000u));
}
template <typename T>
__device__ __forceinline__ void store2(T* p, float a, float b);
template <>
__device__ __forceinline__ void store2<float>(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
template <>
__device__ __forceinline__ void store2<__nv_bfloat16>(__nv_bfloat16* p, float a, float b) {
  const __nv_bfloat162 pair = __floats2bfloat162_rn(a, b);
  *reinterpret_cast<uint32_t*>(p) = *reinterpret_cast<const uint32_t*>(&pair);
}

// The prompts' form: a run of kRun tokens of one sequence.  A lane takes two neighbouring channels (and the two that
// they turn with): all inputs of the run, and the taps - 1 before it, are on their way before the first is used.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kConvWarps * 32) conv_rotary_prep_run_kernel(ConvPrepParams p) {
  extern __shared__ __align__(16) float2 turn[];
  __shared__ TokenInfo infos[kRun];
  __shared__ int64_t cache_rows[kRun];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int NH = p.num_heads, NKV = p.num_kv_heads, D = p.head_dim, DV = p.v_dim, half = p.rotary_dims / 2;
  const int64_t token0 = (int64_t)blockIdx.x * kRun;
  const int run = (int)(p.num_tokens - token0 < kRun ? p.num_tokens - token0 : kRun);
  run_prologue(p, token0, run, infos, cache_rows, turn);
  constexpr int kKeep = TAPS - 1;
  // the channel pair c of the run: u[0 .. kKeep) before the run, then the run's own
  auto inputs = [&](int c, float2 (&u)[kKeep + kRun]) {
    const T* x = (const T*)p.x + c;
    float2 bias = make_float2(0.f, 0.f);
    if (p.bias != nullptr) bias = *reinterpret_cast<const float2*>(p.bias + c);
#pragma unroll
    for (int t = 0; t < kRun; ++t) {
      u[kKeep + t] = make_float2(0.f, 0.f);
      if (t < run) u[kKeep + t] = load2<T>(x + (token0 + t) * p.x_stride);
    }
    const TokenInfo info = infos[0];
#pragma unroll
    for (int j = 0; j < kKeep; ++j) {
      const int back = info.offset - kKeep + j;
      u[j] = make_float2(0.f, 0.f);
      if (back >= 0) {
        u[j] = load2<T>(x + (info.first + back) * p.x_stride);
        u[j].x += bias.x;
        u[j].y += bias.y;
      } else if (info.slot >= 0) {
        const float* before = p.state + (int64_t)info.slot * p.state_stride + p.tail_off + (int64_t)(kKeep + back) * p.channels + c;
        u[j] = make_float2(before[0], before[1]);
      }
    }
#pragma unroll
    for (int t = 0; t < kRun; ++t) {
      u[kKeep + t].x += bias.x;
      u[kKeep + t].y += bias.y;
    }
  };
  auto taps_of = [&](int c, float2 (&w)[TAPS]) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = make_float2(p.conv[(int64_t)c * TAPS + j], p.conv[(int64_t)(c + 1) * TAPS + j]);
  };
  // the inputs that the convolution of the run's token t sees: a token that is its sequence's first (or one of the
  // first few) has zeros, or what its own slot holds, in place of another sequence's inputs
  auto convolve = [&](const float2 (&u)[kKeep + kRun], const float2 (&w)[TAPS], int t, int c) -> float2 {
    float2 y = make_float2(0.f, 0.f);
    const TokenInfo info = infos[t];
    const int own = info.offset < t ? info.offset : t;          // inputs of this sequence inside the run before t
    if (own == t || own >= kKeep) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        y.x = fmaf(w[j].x, u[t + j].x, y.x);
        y.y = fmaf(w[j].y, u[t + j].y, y.y);
      }
      return y;
    }
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int back = info.offset - kKeep + j;
      float2 v = make_float2(0.f, 0.f);
      if (back >= 0) {
        v = u[t + j];
      } else if (info.slot >= 0) {
        const float* before = p.state + (int64_t)info.slot * p.state_stride + p.tail_off + (int64_t)(kKeep + back) * p.channels + c;
        v = make_float2(before[0], before[1]);
      }
      y.x = fmaf(w[j].x, v.x, y.x);
      y.y = fmaf(w[j].y, v.y, y.y);
    }
    return y;
  };
  for (int h = blockIdx.y * kConvWarps + warp; h < NH + 2 * NKV; h += gridDim.y * kConvWarps) {
    const bool is_q = h < NH, is_v = h >= NH + NKV;
    const int g = is_q ? h : (is_v ? h - NH - NKV : h - NH);
    const int width = is_v ? DV : D;
    const int first = is_q ? g * D : (is_v ? (NH + NKV) * D + g * DV : NH * D + g * D);
    auto row_of = [&](int t) -> T* {
      if (is_q) return (T*)p.q_out + ((token0 + t) * NH + g) * (int64_t)D;
      if (cache_rows[t] < 0) return nullptr;
      const int64_t row = cache_rows[t] + (int64_t)g * p.page_size;
      return is_v ? (T*)p.v_cache + row * p.v_row_stride : (T*)p.k_cache + row * p.k_row_stride;
    };
    const int turned = is_v ? 0 : half;
    for (int i = 2 * lane; i < turned; i += 64) {
      float2 ua[kKeep + kRun], ub[kKeep + kRun], wa[TAPS], wb[TAPS];
      inputs(first + i, ua);
      inputs(first + half + i, ub);
      taps_of(first + i, wa);
      taps_of(first + half + i, wb);
#pragma unroll
      for (int t = 0; t < kRun; ++t) {
        if (t >= run) break;
        const float2 a = convolve(ua, wa, t, first + i), b = convolve(ub, wb, t, first + half + i);
        const float4 cs = *reinterpret_cast<const float4*>(turn + t * half + i);       // cos, sin of two pairs
        T* dst = row_of(t);
        if (dst != nullptr) {
          store2<T>(dst + i, a.x * cs.x - b.x * cs.y, a.y * cs.z - b.y * cs.w);
          store2<T>(dst + half + i, b.x * cs.x + a.x * cs.y, b.y * cs.z + a.y * cs.w);
        }
      }
    }
    for (int d = 2 * turned + 2 * lane; d < width; d += 64) {
      float2 u[kKeep + kRun], w[TAPS];
      inputs(first + d, u);
      taps_of(first + d, w);
#pragma unroll
      for (int t = 0; t < kRun; ++t) {
        if (t >= run) break;
        const float2 y = convolve(u, w, t, first + d);
        T* dst = row_of(t);
        if (dst != nullptr) store2<T>(dst + d, y.x, y.y);
      }
    }
  }
}

// whether every pair of channels the runs' form reads and writes at once starts on a boundary of its size
template <typename T>
bool conv_runs_take(const ConvPrepParams& p) {
  auto even = [](int64_t v) { return v % 2 == 0; };
  auto placed = [](const void* q, int bytes) { return reinterpret_cast<uintptr_t>(q) % bytes == 0; };
  const int pair = 2 * (int)sizeof(T);
  return p.layout == 0 && p.taps <= 4 && even(p.rotary_dims / 2) && even(p.head_dim) && even(p.v_dim) && even(p.x_stride) &&
         even(p.k_row_stride) && even(p.v_row_stride) && placed(p.x, pair) && placed(p.q_out, pair) && placed(p.k_cache, pair) &&
         placed(p.v_cache, pair) && placed(p.bias, 8);
}

template <typename T>
int launch_conv_prep_typed(const ConvPrepParams& p, cudaStream_t stream) {
  ConvPrepParams q = p;
  // few tokens: a block per token and as many blocks per token as there are groups of heads
  const int heads = p.num_heads + 2 * p.num_kv_heads;
  q.run = p.num_tokens < 256 || p.keep_tail ? 1 : kRun;
  int across = 1;
  const int64_t runs = (p.num_tokens + q.run - 1) / q.run;
  if (q.run == kRun && conv_runs_take<T>(p)) {
    const dim3 grid((unsigned)runs, (unsigned)((heads + 2 * kConvWarps - 1) / (2 * kConvWarps))), block(kConvWarps * 32);
    const size_t smem = (size_t)kRun * (p.rotary_dims / 2) * sizeof(float2);
    if (runs > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
    switch (p.taps) {
      case 1: return (int)launch_chain(conv_rotary_prep_run_kernel<T, 1>, grid, block, smem, stream, dim3(1, 1, 1), q);
      case 2: return (int)launch_chain(conv_rotary_prep_run_kernel<T, 2>, grid, block, smem, stream, dim3(1, 1, 1), q);
      case 3: return (int)launch_chain(conv_rotary_prep_run_kernel<T, 3>, grid, block, smem, stream, dim3(1, 1, 1), q);
      default: return (int)launch_chain(conv_rotary_prep_run_kernel<T, 4>, grid, block, smem, stream, dim3(1, 1, 1), q);
    }
  }
  while (across < 16 && runs * across < 512 && heads > across * kConvWarps) across *= 2;
  if (runs > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  const dim3 grid((unsigned)runs, (unsigned)across), block(kConvWarps * 32);
  const size_t smem = (size_t)q.run * (p.rotary_dims / 2) * sizeof(float2);
  switch (p.taps) {
    case 1: return (int)launch_chain(conv_rotary_prep_kernel<T, 1>, grid, block, smem, stream, dim3(1, 1, 1), q);
    case 2: return (int)launch_chain(conv_rotary_prep_kernel<T, 2>, grid, block, smem, stream, dim3(1, 1, 1), q);
    case 3: return (int)launch_chain(conv_rotary_prep_kernel<T, 3>, grid, block, smem, stream, dim3(1, 1, 1), q);
    case 4: return (int)launch_chain(conv_rotary_prep_kernel<T, 4>, grid, block, smem, stream, dim3(1, 1, 1), q);
    default:
      return (int)launch_chain(conv_rotary_prep_kernel<T, kConvMaxTaps>, grid, block, smem, stream, dim3(1, 1, 1), q);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) gate_columns_kernel(const T* __restrict__ in, const T* __restrict__ x,
                                                           T* __restrict__ out, int64_t total, int width,
                                                           int64_t x_stride, int64_t out_stride, float factor, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = (blockIdx.x * (int64_t)blockDim.x + threadIdx.x) * (vec ? 8 : 1);
  if (i >= total) return;
  const int64_t token = i / width;
  const int c = (int)(i - token * width);
  const T* gate = x + token * x_stride + c;
  T* dst = out + token * out_stride + c;
  if (!vec) {
    dst[0] = from_float<T>(to_float<T>(in[i]) * factor / (1.f + expf(-to_float<T>(gate[0]))));
    return;
  }
  float v[8], g[8];
  load8<T>(in + i, v);
  load8<T>(gate, g);
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] = v[e] * factor / (1.f + expf(-g[e]));
  if constexpr (sizeof(T) == 2) {
    uint4 packed;
    uint32_t* w = reinterpret_cast<uint32_t*>(&packed);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const __nv_bfloat162 pair = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
      w[e] = *reinterpret_cast<const uint32_t*>(&pair);
    }
    *reinterpret_cast<uint4*>(dst) = packed;
  } else {
    *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(dst + 4) = make_float4(v[4], v[5], v[6], v[7]);
  }
}

template <typename T>
int launch_gate_typed(const void* in, const void* x, void* out, int64_t tokens, int width, int64_t x_stride,
                      int64_t out_stride, float factor, cudaStream_t stream) {
  const int64_t total = tokens * width;
  constexpr int per16 = 16 / (int)sizeof(T);
  const int vec = width % 8 == 0 && x_stride % per16 == 0 && out_stride % per16 == 0 &&
                  (reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out)) % 16 == 0;
  const int64_t blocks = (total / (vec ? 8 : 1) + 255) / 256;
  if (blocks > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  return (int)launch_chain(gate_columns_kernel<T>, dim3((unsigned)blocks), dim3(256), 0, stream, dim3(1, 1, 1),
                           (const T*)in, (const T*)x, (T*)out, total, width, x_stride, out_stride, factor, vec);
}

}  // namespace

int launch_conv_rotary_prep(const ConvPrepParams& p, cudaStream_t stream) {
  if (p.num_tokens == 0) return 0;
  if (p.rotary_dims < 0 || p.rotary_dims % 2 || p.rotary_dims > p.head_dim || p.rotary_dims > 1024 || p.taps < 1 ||
      p.taps > kConvMaxTaps || p.num_seqs < 1 || (p.layout != 0 && p.layout != 1) || (p.taps > 1 && p.state == nullptr))
    return (int)cudaErrorInvalidValue;
  return p.dtype == kBFloat16 ? launch_conv_prep_typed<__nv_bfloat16>(p, stream) : launch_conv_prep_typed<float>(p, stream);
}

int launch_gate_columns(const void* in, const void* x, void* out, int64_t tokens, int width, int64_t x_stride,
                        int64_t out_stride, float factor, int dtype, cudaStream_t stream) {
  if (tokens == 0 || width == 0) return 0;
  return dtype == kBFloat16 ? launch_gate_typed<__nv_bfloat16>(in, x, out, tokens, width, x_stride, out_stride, factor, stream)
                            : launch_gate_typed<float>(in, x, out, tokens, width, x_stride, out_stride, factor, stream);
}

}  // namespace akv
