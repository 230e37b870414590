// Layers whose branches are normed on the way in and on the way out: what stands between one branch's result and the
// next branch's input is one kernel.
//
//   hidden += b / sqrt(mean(b^2) + eps) * weight                      b: the branch's result
//   out     = hidden / sqrt(mean(hidden^2) + next_eps) * next_weight
//
// b is a stored row, or the rows of routed experts that are still to be added up: a token's `top` float32 rows in the
// order of its choices (plus a shared expert's row), where a choice that is the identity counts as its weight times the
// token's input row and has no row of its own.
//
// A block per (row, slice of the columns); on few rows the blocks of a row form a cluster that shares the columns and
// adds up both sums of squares through distributed shared memory in rank order.  The slice stays in shared memory
// between the passes.  Everything is float; 16-byte accesses where every row and operand allows them.
#include <algorithm>

#include "common.cuh"
#include "launchers.h"

namespace akv {

namespace {

template <int VEC>
__device__ __forceinline__ void load_f32(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  } else {
    v[0] = *p;
  }
}
template <int VEC>
__device__ __forceinline__ void load_any(const void* base, int dtype, int64_t i, float (&v)[VEC]) {
  if (dtype != kBFloat16) {
    load_f32<VEC>((const float*)base + i, v);
    return;
  }
  const __nv_bfloat16* p = (const __nv_bfloat16*)base + i;
  if constexpr (VEC == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(raw.x << 16); v[1] = __uint_as_float(raw.x & 0xffff0000u);
    v[2] = __uint_as_float(raw.y << 16); v[3] = __uint_as_float(raw.y & 0xffff0000u);
  } else {
    v[0] = __bfloat162float(*p);
  }
}
template <int VEC>
__device__ __forceinline__ void store_f32(float* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int VEC>
__device__ __forceinline__ void store_any(void* base, int dtype, int64_t i, const float (&v)[VEC]) {
  if (dtype != kBFloat16) {
    store_f32<VEC>((float*)base + i, v);
    return;
  }
  __nv_bfloat16* p = (__nv_bfloat16*)base + i;
  if constexpr (VEC == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<const uint32_t*>(&a);
    raw.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

}  // namespace

template <int VEC>
__global__ void __launch_bounds__(256) branch_rmsnorm_kernel(BranchNormParams p, int chunk) {
  extern __shared__ __align__(16) float slice[];
  __shared__ float scratch[34];
  __shared__ int own_row[kBranchNormMaxTop];         // the choices that have a row of their own, in their order
  __shared__ int own_rows;
  __shared__ float identity_weight;                  // the sum of the other choices' weights, in their order
  pdl_launch_dependents();
  pdl_wait();
  const int W = p.width;
  int64_t token = blockIdx.x;
  bool bad = false;
  if (p.rows != nullptr) {
    token = p.rows[blockIdx.x];
    if (token < 0 || token >= p.num_tokens) {        // every block of the row sees the same: they skip together
      if (threadIdx.x == 0) set_status(p.status, kBadRow);
      bad = true;
      token = 0;
    }
  }
  const bool routed = p.branch == nullptr;
  if (routed) {
    if (threadIdx.x == 0) {
      float sum = 0.f;
      int own = 0;
      for (int s = 0; s < p.top; ++s) {
        if (p.chosen == nullptr || p.chosen[token * p.top + s] < p.first_identity) own_row[own++] = s;
        else sum += p.pair_weights[token * p.top + s];
      }
      own_rows = own;
      identity_weight = sum;
    }
    __syncthreads();
  }
  const int rows_here = routed ? own_rows : 0;
  const int c0 = blockIdx.y * chunk, c1 = bad ? c0 : min(W, c0 + chunk);
  const int step = blockDim.x * VEC;
  float ss = 0.f;
  for (int c = c0 + threadIdx.x * VEC; c < c1; c += step) {
    float v[VEC];
    if (!routed) {
      load_any<VEC>(p.branch, p.branch_dtype, token * W + c, v);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = 0.f;
#pragma unroll 4
      for (int s = 0; s < rows_here; ++s) {
        float r[VEC];
        load_f32<VEC>(p.parts + (token * p.top + own_row[s]) * W + c, r);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] += r[e];
      }
      if (p.chosen != nullptr && identity_weight != 0.f) {
        float r[VEC];
        load_any<VEC>(p.x, p.x_dtype, token * W + c, r);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = fmaf(identity_weight, r[e], v[e]);
      }
      if (p.shared != nullptr) {
        float r[VEC];
        load_any<VEC>(p.shared, p.shared_dtype, token * W + c, r);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] += r[e];
      }
    }
    store_f32<VEC>(slice + (c - c0), v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(v[e], v[e], ss);
  }
  ss = cluster_sum(ss, scratch);
  const float inv = 1.f / sqrtf(ss / (float)W + p.eps);
  float* hidden = p.hidden + token * W;
  ss = 0.f;
  for (int c = c0 + threadIdx.x * VEC; c < c1; c += step) {      // a thread meets the columns it stored
    float v[VEC], w[VEC], h[VEC];
    load_f32<VEC>(slice + (c - c0), v);
    load_f32<VEC>(p.weight + c, w);
    load_f32<VEC>(hidden + c, h);
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      h[e] += v[e] * inv * w[e];
      ss = fmaf(h[e], h[e], ss);
    }
    if (p.rows == nullptr) store_f32<VEC>(hidden + c, h);
    if (p.out != nullptr) store_f32<VEC>(slice + (c - c0), h);
  }
  if (p.out == nullptr) return;                                  // the same for every block of the cluster
  ss = cluster_sum(ss, scratch);
  const float next_inv = 1.f / sqrtf(ss / (float)W + p.next_eps);
  for (int c = c0 + threadIdx.x * VEC; c < c1; c += step) {
    float v[VEC], w[VEC];
    load_f32<VEC>(slice + (c - c0), v);
    load_f32<VEC>(p.next_weight + c, w);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] *= next_inv * w[e];
    store_any<VEC>(p.out, p.out_dtype, (int64_t)blockIdx.x * W + c, v);
  }
}

int launch_branch_rmsnorm(const BranchNormParams& p, cudaStream_t stream) {
  const int64_t blocks = p.rows != nullptr ? p.num_rows : p.num_tokens;
  if (blocks == 0) return 0;
  if (p.width < 1 || blocks > 0x7fffffffLL || p.weight == nullptr || (p.branch == nullptr) == (p.parts == nullptr) ||
      (p.parts != nullptr && (p.top < 1 || p.top > kBranchNormMaxTop)) ||
      (p.chosen != nullptr && (p.pair_weights == nullptr || p.x == nullptr)) ||
      (p.out == nullptr) != (p.next_weight == nullptr) || (p.rows != nullptr && p.out == nullptr))
    return (int)cudaErrorInvalidValue;
  auto aligned = [](const void* ptr) { return reinterpret_cast<uintptr_t>(ptr) % 16 == 0; };
  const bool wide = p.width % 4 == 0 && aligned(p.hidden) && aligned(p.branch) && aligned(p.parts) && aligned(p.shared) &&
                    aligned(p.x) && aligned(p.weight) && aligned(p.next_weight) && aligned(p.out);
  const int vec = wide ? 4 : 1;
  const int parts = row_cluster(blocks, p.width);
  const int chunk = ((p.width / vec + parts - 1) / parts) * vec;
  const size_t smem = (size_t)chunk * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  auto kernel = wide ? branch_rmsnorm_kernel<4> : branch_rmsnorm_kernel<1>;
  if (smem > 48 * 1024) {
    cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
  }
  const int threads = std::min(256, std::max(32, (chunk / vec + 31) / 32 * 32));
  return (int)launch_chain(kernel, dim3((unsigned)blocks, (unsigned)parts), dim3(threads), smem, stream,
                           dim3(1, parts, 1), p, chunk);
}

}  // namespace akv
