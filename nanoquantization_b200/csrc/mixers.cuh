// Helpers shared by the sequence-mixing kernels: element types and the flattened-batch descriptor.
#pragma once
#include "common.cuh"
#include "nqb200_mixers.h"

namespace nqb200 {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_f(float v) { return 1.f / (1.f + expf(-v)); }
// log(sigmoid(v)), right at both ends
__device__ __forceinline__ float log_sigmoid_f(float v) { return fminf(v, 0.f) - log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float gelu_erf_f(float v) { return 0.5f * v * (1.f + erff(v * 0.70710678118654752f)); }
__device__ __forceinline__ float gelu_tanh_f(float v) {
  return 0.5f * v * (1.f + tanhf(0.79788456080286536f * (v + 0.044715f * v * v * v)));
}

// For bf16 results: a few float ulps, out of the hardware's exponential and reciprocal.
__device__ __forceinline__ float ex2_fast(float x) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }
__device__ __forceinline__ float rcp_fast(float x) { float r; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }
__device__ __forceinline__ float sigmoid_fast(float v) { return rcp_fast(1.f + ex2_fast(v * -1.4426950408889634f)); }
__device__ __forceinline__ float exp_fast(float v) { return ex2_fast(v * 1.4426950408889634f); }
// tanh as 1 - 2 / (1 + e^2y): absolute error of a few 1e-7, right at both ends
__device__ __forceinline__ float tanh_fast(float y) { return 1.f - 2.f * rcp_fast(1.f + ex2_fast(y * 2.8853900817779268f)); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xFFFFFFFFu, v, o));
  return v;
}

// Cache row of position p of sequence b.
__device__ __forceinline__ size_t kv_row(const nqb200_batch& bt, int b, int p) {
  return (size_t)bt.table[(size_t)b * bt.table_width + p / bt.block_size] * bt.block_size + p % bt.block_size;
}

// mixer_attention_umma.cu: attention of prompts with tcgen05.
bool attention_umma_supports(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, const void* out, int64_t out_stride,
                             int64_t cache_rows, const nqb200_attention* a, const nqb200_batch* b);
int attention_umma(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, void* out, int64_t out_stride, int64_t cache_rows,
                   const nqb200_attention* a, const nqb200_batch* b, int* status, cudaStream_t st);
// mixer_prefill.cu: the same for the sizes and pages that kernel does not take, and for short portions.
bool attention_prefill_supports(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, const void* out, int64_t out_stride,
                                const nqb200_attention* a);
int attention_prefill(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, void* out, int64_t out_stride,
                      const nqb200_attention* a, const nqb200_batch* b, cudaStream_t st);

static inline int check_batch(const nqb200_batch* b, bool paged) {
  if (!b) return NQB200_ERR_NULL_POINTER;
  if (b->batch < 0 || b->tokens < 0 || b->max_len < 0 || b->max_len > b->tokens || b->batch > 65535) return NQB200_ERR_BAD_SHAPE;
  if (b->tokens == 0) return NQB200_OK;
  if (b->batch == 0 || b->max_len == 0) return NQB200_ERR_BAD_SHAPE;
  if (!b->cu || !b->pos0) return NQB200_ERR_NULL_POINTER;
  if (paged ? (!b->table || b->table_width <= 0 || b->block_size <= 0) : !b->slot) return NQB200_ERR_NULL_POINTER;
  return NQB200_OK;
}
static inline bool mixer_dtype(int dtype) { return dtype == NQB200_BF16 || dtype == NQB200_F32; }

}  // namespace nqb200
