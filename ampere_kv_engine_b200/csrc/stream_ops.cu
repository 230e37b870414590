// Small kernels on the float32 residual stream and on branch outputs:
//
//   pair_rows_add   hidden[t] += table[(prev(t) * mul_prev + token(t) * mul_cur) mod buckets], and row `buckets` for a
//                   sequence's first token (position 0).  prev(t) is the token before t in the same sequence: the row
//                   above inside a step, and for a step's first row the last token of the step before, which the
//                   request keeps in its state slot (one int32).  The block of a sequence's first row reads that
//                   token and then stores the sequence's newest one; no other block touches the slot.
//   stream_add      hidden += other (both float32)
//   scaled_sum      out = a * sa + b * sb, formed in float32 and rounded once
//   stream_sum      hidden += the results of several branches at once (tensors, or the experts' rows of a token still to
//                   be added up), and a rounded copy of the new stream for a product that reads the stream itself
//   stream_concat   [hidden | start], rounded, for a product that reads the stream beside what it was at the start
//   stream_row_add  hidden += one row, the same for every token
//   token_gate      gelu_tanh(z) * (a part of the row that the token's id picks from a table)
#include "common.cuh"
#include "launchers.h"

namespace akv {

namespace {

__device__ __forceinline__ int64_t resolve_token(int64_t id, const int32_t* sampled, int64_t num_sampled, int64_t vocab) {
  if (id < 0 && sampled != nullptr && -id - 1 < num_sampled) id = sampled[-id - 1];
  return (id < 0 || id >= vocab) ? 0 : id;             // the embedding kernel has reported it
}

template <typename T>
__global__ void pair_rows_add_kernel(PairRowsParams p) {
  __shared__ int64_t prev_shared;
  pdl_launch_dependents();
  pdl_wait();
  const int64_t token = blockIdx.x;
  // the sequence whose rows hold this token: the last s with cu_q[s] <= token
  int lo = 0, hi = p.num_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.cu_q[mid] <= token) lo = mid;
    else hi = mid - 1;
  }
  const int seq = lo;
  const bool first_row = token == p.cu_q[seq];
  const int slot = p.state_slots[seq];
  const int64_t cur = resolve_token(p.ids[token], p.sampled, p.num_sampled, p.vocab);
  if (threadIdx.x == 0) {
    int64_t prev = 0;
    if (!first_row) prev = resolve_token(p.ids[token - 1], p.sampled, p.num_sampled, p.vocab);
    else if (slot >= 0) prev = p.last_token[(int64_t)slot * p.state_stride];
    prev_shared = prev;
    if (first_row && slot >= 0) {
      const int64_t last = p.cu_q[seq + 1] - 1;
      if (last >= token && last < p.num_tokens)
        p.last_token[(int64_t)slot * p.state_stride] =
            (int32_t)resolve_token(p.ids[last], p.sampled, p.num_sampled, p.vocab);
    }
  }
  __syncthreads();
  int64_t row = p.buckets;
  if (p.positions[token] > 0) {
    row = (prev_shared * p.mul_prev + cur * p.mul_cur) % p.buckets;
    if (row < 0) row += p.buckets;
  }
  const T* src = (const T*)p.table + row * p.hidden_size;
  float* dst = p.hidden + token * p.hidden_size;
  for (int64_t i = threadIdx.x; i < p.hidden_size; i += blockDim.x) dst[i] += to_float<T>(src[i]);
}

__global__ void stream_add_kernel(float* __restrict__ hidden, const float* __restrict__ other, int64_t n) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = (blockIdx.x * (int64_t)blockDim.x + threadIdx.x) * 4;
  if (i + 3 < n) {
    float4 a = *reinterpret_cast<float4*>(hidden + i);
    const float4 b = *reinterpret_cast<const float4*>(other + i);
    a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w;
    *reinterpret_cast<float4*>(hidden + i) = a;
  } else {
    for (int64_t k = i; k < n; ++k) hidden[k] += other[k];
  }
}

template <typename T>
__global__ void scaled_sum_kernel(const T* __restrict__ a, const T* __restrict__ b, T* __restrict__ out, float sa,
                                  float sb, int64_t n) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x;
  if (i < n) out[i] = from_float<T>(to_float<T>(a[i]) * sa + to_float<T>(b[i]) * sb);
}

// four elements from column c of a row in either dtype
__device__ __forceinline__ float4 load4_any(const void* p, int64_t i, int dtype) {
  if (dtype == kBFloat16) {
    const uint2 raw = *reinterpret_cast<const uint2*>((const __nv_bfloat16*)p + i);
    return make_float4(__uint_as_float(raw.x << 16), __uint_as_float(raw.x & 0xffff0000u), __uint_as_float(raw.y << 16),
                       __uint_as_float(raw.y & 0xffff0000u));
  }
  return *reinterpret_cast<const float4*>((const float*)p + i);
}
__device__ __forceinline__ float load_one(const void* p, int64_t i, int dtype) {
  return dtype == kBFloat16 ? __bfloat162float(((const __nv_bfloat16*)p)[i]) : ((const float*)p)[i];
}
__device__ __forceinline__ void add4(float4& a, const float4& b) { a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w; }
__device__ __forceinline__ void store4_bf16(void* p, int64_t i, const float4& v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>((__nv_bfloat16*)p + i) =
      make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

// four columns a thread where the width allows it (vec), else one
__global__ void __launch_bounds__(256) stream_sum_kernel(StreamSumParams p, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = (blockIdx.x * (int64_t)blockDim.x + threadIdx.x) * (vec ? 4 : 1);
  if (i >= p.num_tokens * p.width) return;
  const int64_t token = i / p.width;
  const int c = (int)(i - token * p.width);
  if (vec) {
    float4 h = *reinterpret_cast<float4*>(p.hidden + i);
    if (p.a != nullptr) add4(h, load4_any(p.a, i, p.a_dtype));
    if (p.b != nullptr) add4(h, load4_any(p.b, i, p.b_dtype));
    if (p.parts != nullptr) {
      float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int s = 0; s < p.top; ++s)
        add4(sum, *reinterpret_cast<const float4*>(p.parts + (token * p.top + s) * p.width + c));
      if (p.shared != nullptr) add4(sum, load4_any(p.shared, i, p.shared_dtype));
      add4(h, sum);
    }
    *reinterpret_cast<float4*>(p.hidden + i) = h;
    if (p.copy != nullptr) {
      if (p.copy_dtype == kBFloat16) store4_bf16(p.copy, i, h);
      else *reinterpret_cast<float4*>((float*)p.copy + i) = h;
    }
    return;
  }
  float h = p.hidden[i];
  if (p.a != nullptr) h += load_one(p.a, i, p.a_dtype);
  if (p.b != nullptr) h += load_one(p.b, i, p.b_dtype);
  if (p.parts != nullptr) {
    float sum = 0.f;
    for (int s = 0; s < p.top; ++s) sum += p.parts[(token * p.top + s) * p.width + c];
    if (p.shared != nullptr) sum += load_one(p.shared, i, p.shared_dtype);
    h += sum;
  }
  p.hidden[i] = h;
  if (p.copy != nullptr) {
    if (p.copy_dtype == kBFloat16) ((__nv_bfloat16*)p.copy)[i] = __float2bfloat16_rn(h);
    else ((float*)p.copy)[i] = h;
  }
}

template <typename T>
__global__ void __launch_bounds__(256) stream_concat_kernel(const float* __restrict__ hidden, const float* __restrict__ start,
                                                            T* __restrict__ out, int64_t total, int width, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = (blockIdx.x * (int64_t)blockDim.x + threadIdx.x) * (vec ? 4 : 1);     // an element of out
  if (i >= total) return;
  const int64_t token = i / (2 * width);
  const int c = (int)(i - token * 2 * width);
  const float* src = c < width ? hidden + token * width + c : start + token * width + (c - width);
  if (!vec) {
    out[i] = from_float<T>(*src);
    return;
  }
  const float4 v = *reinterpret_cast<const float4*>(src);
  if constexpr (sizeof(T) == 2) store4_bf16(out, i, v);
  else *reinterpret_cast<float4*>(out + i) = v;
}

__global__ void __launch_bounds__(256) stream_row_add_kernel(float* __restrict__ hidden, const float* __restrict__ row,
                                                             int64_t total, int width, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = (blockIdx.x * (int64_t)blockDim.x + threadIdx.x) * (vec ? 4 : 1);
  if (i >= total) return;
  const int c = (int)(i % width);
  if (!vec) {
    hidden[i] += row[c];
    return;
  }
  float4 h = *reinterpret_cast<float4*>(hidden + i);
  add4(h, *reinterpret_cast<const float4*>(row + c));
  *reinterpret_cast<float4*>(hidden + i) = h;
}

// The tanh form of GELU as z / (1 + e^(-2u)), (1 + tanh u) / 2 being 1 / (1 + e^(-2u)): what leaves here is divided by its
// own root mean square later, so it keeps its relative precision far below zero too.
__device__ __forceinline__ float gelu_tanh_tail(float z) {
  return z / (1.f + expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
}

template <typename T>
__global__ void token_gate_kernel(TokenGateParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t token = blockIdx.x;
  int64_t id = p.ids[token];
  if (id < 0 && p.sampled != nullptr && -id - 1 < p.num_sampled) id = p.sampled[-id - 1];
  if (id < 0 || id >= p.vocab) {
    if (threadIdx.x == 0) set_status(p.status, kBadToken);
    id = 0;
  }
  const T* e = (const T*)p.table + id * p.table_stride + p.col_off;
  const T* z = (const T*)p.z + token * p.dim;
  T* out = (T*)p.out + token * p.dim;
  for (int c = threadIdx.x; c < p.dim; c += blockDim.x)
    out[c] = from_float<T>(gelu_tanh_tail(to_float<T>(z[c])) * to_float<T>(e[c]));
}

bool aligned16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

}  // namespace

int launch_stream_sum(const StreamSumParams& p, cudaStream_t stream) {
  const int64_t total = p.num_tokens * p.width;
  if (total == 0) return 0;
  const int vec = p.width % 4 == 0 && aligned16(p.hidden) && aligned16(p.a) && aligned16(p.b) && aligned16(p.parts) &&
                  aligned16(p.shared) && aligned16(p.copy);
  const int64_t blocks = ((vec ? total / 4 : total) + 255) / 256;
  if (blocks > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  return (int)launch_chain(stream_sum_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, dim3(1, 1, 1), p, vec);
}

int launch_stream_concat(const float* hidden, const float* start, void* out, int64_t num_tokens, int width, int dtype,
                         cudaStream_t stream) {
  const int64_t total = num_tokens * 2 * width;
  if (total == 0) return 0;
  const int vec = width % 4 == 0 && aligned16(hidden) && aligned16(start) && aligned16(out);
  const int64_t blocks = ((vec ? total / 4 : total) + 255) / 256;
  if (blocks > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  if (dtype == kBFloat16)
    return (int)launch_chain(stream_concat_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, stream,
                             dim3(1, 1, 1), hidden, start, (__nv_bfloat16*)out, total, width, vec);
  return (int)launch_chain(stream_concat_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream, dim3(1, 1, 1), hidden,
                           start, (float*)out, total, width, vec);
}

int launch_stream_row_add(float* hidden, const float* row, int64_t num_tokens, int width, cudaStream_t stream) {
  const int64_t total = num_tokens * width;
  if (total == 0) return 0;
  const int vec = width % 4 == 0 && aligned16(hidden) && aligned16(row);
  const int64_t blocks = ((vec ? total / 4 : total) + 255) / 256;
  if (blocks > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  return (int)launch_chain(stream_row_add_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, dim3(1, 1, 1), hidden, row,
                           total, width, vec);
}

int launch_token_gate(const TokenGateParams& p, cudaStream_t stream) {
  if (p.num_tokens == 0 || p.dim == 0) return 0;
  if (p.num_tokens > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  const int threads = p.dim >= 256 ? 256 : (p.dim + 31) / 32 * 32;
  if (p.dtype == kBFloat16)
    return (int)launch_chain(token_gate_kernel<__nv_bfloat16>, dim3((unsigned)p.num_tokens), dim3(threads), 0, stream,
                             dim3(1, 1, 1), p);
  return (int)launch_chain(token_gate_kernel<float>, dim3((unsigned)p.num_tokens), dim3(threads), 0, stream, dim3(1, 1, 1), p);
}

int launch_pair_rows_add(const PairRowsParams& p, cudaStream_t stream) {
  if (p.num_tokens == 0) return 0;
  if (p.buckets < 1 || p.num_seqs < 1) return (int)cudaErrorInvalidValue;
  const int threads = (int)(p.hidden_size >= 1024 ? 256 : (p.hidden_size >= 128 ? 128 : 32));
  if (p.dtype == kBFloat16)
    return (int)launch_chain(pair_rows_add_kernel<__nv_bfloat16>, dim3((unsigned)p.num_tokens), dim3(threads), 0, stream,
                             dim3(1, 1, 1), p);
  return (int)launch_chain(pair_rows_add_kernel<float>, dim3((unsigned)p.num_tokens), dim3(threads), 0, stream,
                           dim3(1, 1, 1), p);
}

int launch_stream_add(float* hidden, const float* other, int64_t n, cudaStream_t stream) {
  if (n == 0) return 0;
  const int64_t blocks = ((n + 3) / 4 + 255) / 256;
  if (blocks > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  return (int)launch_chain(stream_add_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, dim3(1, 1, 1), hidden, other, n);
}

int launch_scaled_sum(const void* a, const void* b, void* out, float sa, float sb, int64_t n, int dtype,
                      cudaStream_t stream) {
  if (n == 0) return 0;
  const int64_t blocks = (n + 255) / 256;
  if (blocks > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  if (dtype == kBFloat16)
    return (int)launch_chain(scaled_sum_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, stream, dim3(1, 1, 1),
                             (const __nv_bfloat16*)a, (const __nv_bfloat16*)b, (__nv_bfloat16*)out, sa, sb, n);
  return (int)launch_chain(scaled_sum_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream, dim3(1, 1, 1),
                           (const float*)a, (const float*)b, (float*)out, sa, sb, n);
}

}  // namespace akv
