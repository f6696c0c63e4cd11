// Routing: a warp per token takes the scores, the groups and the experts; then the pairs are sorted by expert.  Few tokens:
// one CTA does all of it.  Many: the routing CTAs count, one CTA scans the counts, and the pairs are dealt to their places.
#include <limits.h>
#include "moe.cuh"

namespace nqb200 {

constexpr int kRouteMaxExperts = 1024;      // 32 per lane
constexpr int kRouteSmallTokens = 32;

// Floats (no NaN) as integers in the same order, above 0.
__device__ __forceinline__ uint32_t ordered(float v) {
  const uint32_t u = __float_as_uint(v + 0.f);
  return (u >> 31) ? ~u : u | 0x80000000u;
}
// Index of the largest open key (bit i of a lane's mask: item lane + 32 i), the lowest index among equals.
__device__ __forceinline__ int warp_argmax(const uint32_t* key, uint32_t open, int lane) {
  uint32_t best = 0;
  int at = INT_MAX;
  while (open) {
    const int i = __ffs(open) - 1, e = lane + 32 * i;
    open &= open - 1;
    if (key[e] > best) { best = key[e]; at = e; }
  }
  const uint32_t top = __reduce_max_sync(0xFFFFFFFFu, best);
  return __reduce_min_sync(0xFFFFFFFFu, best == top ? at : INT_MAX);
}

// smem: [experts] scores, [experts] choices, [groups] group scores, all this warp's own.
__device__ void route_token(const float* __restrict__ z, const nqb200_router& r, float* smem, int lane, int32_t* expert, float* weight,
                            int* copy = nullptr) {
  float *s = smem, *choice = s + r.experts;
  uint32_t *key = reinterpret_cast<uint32_t*>(choice), *gs = key + r.experts;   // the choices are keys once the groups have their scores
  for (int e = lane; e < r.experts; e += 32) {
    const float v = sigmoid_f(z[e]);
    s[e] = v;
    const float c = v + (r.correction ? r.correction[e] : 0.f);
    choice[e] = c == c ? c : -INFINITY;    // so that any two compare, and every lane ends with the same expert
  }
  __syncwarp();
  const int size = r.experts / r.groups;
  uint32_t open = 0;
  if (r.keep < r.groups) {
    uint32_t gopen = 0;
    for (int g = lane, i = 0; g < r.groups; g += 32, ++i) {
      float a = choice[g * size], b = -INFINITY;
      for (int k = 1; k < size; ++k) {
        const float v = choice[g * size + k];
        if (v > a) { b = a; a = v; } else if (v > b) { b = v; }
      }
      const float sum = size > 1 ? a + b : a;
      gs[g] = ordered(sum == sum ? sum : -INFINITY);
      gopen |= 1u << i;
    }
    __syncwarp();
    for (int k = 0; k < r.keep; ++k) {
      const int g = warp_argmax(gs, gopen, lane), lo = g * size;
      if (lane == (g & 31)) gopen &= ~(1u << (g >> 5));
      for (int i = 0; lane + 32 * i < r.experts; ++i)
        if (lane + 32 * i >= lo && lane + 32 * i < lo + size) open |= 1u << i;
    }
  } else {
    for (int i = 0; lane + 32 * i < r.experts; ++i) open |= 1u << i;
  }
  for (int e = lane; e < r.experts; e += 32) key[e] = ordered(choice[e]);
  __syncwarp();
  float sum = 0.f;
  int mine[4] = {0, 0, 0, 0};   // of choices lane, lane + 32, ...
  for (int k = 0; k < r.top; ++k) {
    const int e = warp_argmax(key, open, lane);
    if (lane == (e & 31)) open &= ~(1u << (e >> 5));
    sum += s[e];
    if (lane == (k & 31)) mine[(k >> 5) & 3] = e;
  }
  for (int k = lane; k < r.top; k += 32) {
    const int e = mine[(k >> 5) & 3];
    expert[k] = e;
    if (copy) copy[k] = e;
    weight[k] = s[e] / (sum + 1e-20f) * r.scale;
  }
  __syncwarp();
}

// Inclusive sum over the CTA's threads (a multiple of 32, up to 1024); every thread calls it.
__device__ __forceinline__ int block_scan(int v, int* warp_sums) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int u = __shfl_up_sync(0xFFFFFFFFu, v, o);
    if (lane >= o) v += u;
  }
  if (lane == 31) warp_sums[warp] = v;
  __syncthreads();
  int before = 0;
  for (int w = 0; w < warp && w < warps; ++w) before += warp_sums[w];
  __syncthreads();
  return before + v;
}

// Thread e holds expert e's count: offsets, the list of experts with tokens; returns the expert's first place.
__device__ __forceinline__ int place_experts(int count, int experts, const nqb200_moe_plan& p, int* warp_sums) {
  const int e = threadIdx.x, end = block_scan(count, warp_sums), slot = block_scan(count > 0 ? 1 : 0, warp_sums);
  if (e < experts) {
    p.offsets[e] = end - count;
    if (e == experts - 1) { p.offsets[experts] = end; p.active[0] = slot; }
    if (count > 0) p.active[slot] = e;
  }
  return end - count;
}

__global__ void __launch_bounds__(1024) moe_route_small_kernel(const float* __restrict__ logits, const nqb200_router r, const nqb200_moe_plan p, int tokens) {
  extern __shared__ float route_smem[];
  __shared__ int hist[kRouteMaxExperts], warp_sums[32];
  grid_launch_dependents();
  grid_dependency_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pairs = tokens * r.top;
  int* expert = reinterpret_cast<int*>(route_smem);     // [pairs]
  float* scores = route_smem + pairs;
  for (int e = threadIdx.x; e < r.experts; e += blockDim.x) hist[e] = 0;
  if (warp < tokens)
    route_token(logits + (size_t)warp * r.experts, r, scores + (size_t)warp * (2 * r.experts + r.groups), lane, p.expert + warp * r.top, p.weight + warp * r.top,
                expert + warp * r.top);
  __syncthreads();
  for (int q = threadIdx.x; q < pairs; q += blockDim.x) atomicAdd(&hist[expert[q]], 1);
  __syncthreads();
  const int count = (int)threadIdx.x < r.experts ? hist[threadIdx.x] : 0;
  const int first = place_experts(count, r.experts, p, warp_sums);
  if ((int)threadIdx.x < r.experts) hist[threadIdx.x] = first;
  __syncthreads();
  for (int q = threadIdx.x; q < pairs; q += blockDim.x) p.order[atomicAdd(&hist[expert[q]], 1)] = q;
}

constexpr int kRouteWarps = 8;
__global__ void __launch_bounds__(kRouteWarps * 32) moe_route_kernel(const float* __restrict__ logits, const nqb200_router r, const nqb200_moe_plan p,
                                                                     int tokens) {
  extern __shared__ float route_smem[];
  __shared__ int hist[kRouteMaxExperts];
  grid_launch_dependents();
  grid_dependency_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int e = threadIdx.x; e < r.experts; e += blockDim.x) hist[e] = 0;
  __syncthreads();
  const int t = blockIdx.x * kRouteWarps + warp;
  if (t < tokens) {
    int32_t* ex = p.expert + (size_t)t * r.top;
    route_token(logits + (size_t)t * r.experts, r, route_smem + (size_t)warp * (2 * r.experts + r.groups), lane, ex, p.weight + (size_t)t * r.top);
    for (int k = lane; k < r.top; k += 32) atomicAdd(&hist[ex[k]], 1);
  }
  __syncthreads();
  for (int e = threadIdx.x; e < r.experts; e += blockDim.x)
    if (hist[e] > 0) atomicAdd(&p.counters[e], hist[e]);
}

__global__ void __launch_bounds__(1024) moe_scan_kernel(const nqb200_moe_plan p, int experts) {
  __shared__ int warp_sums[32];
  grid_launch_dependents();
  grid_dependency_wait();
  const int e = threadIdx.x, first = place_experts(e < experts ? p.counters[e] : 0, experts, p, warp_sums);
  if (e < experts) p.counters[experts + e] = first;
}

constexpr int kScatterPairs = 8;   // per thread
__global__ void __launch_bounds__(256) moe_scatter_kernel(const nqb200_moe_plan p, int experts, int pairs) {
  __shared__ int hist[kRouteMaxExperts];
  grid_launch_dependents();
  grid_dependency_wait();
  for (int e = threadIdx.x; e < experts; e += 256) hist[e] = 0;
  __syncthreads();
  int ex[kScatterPairs], rank[kScatterPairs];
  const int q0 = blockIdx.x * 256 * kScatterPairs + threadIdx.x;
#pragma unroll
  for (int i = 0; i < kScatterPairs; ++i) {
    const int q = q0 + i * 256;
    ex[i] = q < pairs ? p.expert[q] : -1;
    rank[i] = ex[i] >= 0 ? atomicAdd(&hist[ex[i]], 1) : 0;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < experts; e += 256)
    if (hist[e] > 0) hist[e] = atomicAdd(&p.counters[experts + e], hist[e]);
  __syncthreads();
#pragma unroll
  for (int i = 0; i < kScatterPairs; ++i)
    if (ex[i] >= 0) p.order[hist[ex[i]] + rank[i]] = q0 + i * 256;
}

static bool router_ok(const nqb200_router* r) {
  return r->experts > 0 && r->experts <= kRouteMaxExperts && r->groups > 0 && r->experts % r->groups == 0 && r->keep > 0 && r->keep <= r->groups &&
         r->top > 0 && r->top <= 128 && (int64_t)r->top <= (int64_t)r->keep * (r->experts / r->groups);
}

}  // namespace nqb200

using namespace nqb200;

extern "C" int nqb200_moe_route(const float* logits, const nqb200_router* r, const nqb200_moe_plan* plan, int64_t tokens, void* stream) {
  if (!r || !plan) return NQB200_ERR_NULL_POINTER;
  if (tokens < 0 || !router_ok(r) || tokens * r->top > INT32_MAX) return NQB200_ERR_BAD_SHAPE;
  if (tokens == 0) return NQB200_OK;
  if (!logits || !plan->expert || !plan->weight || !plan->offsets || !plan->order || !plan->active || !plan->counters) return NQB200_ERR_NULL_POINTER;
  cudaStream_t st = (cudaStream_t)stream;
  const size_t per_warp = (size_t)(2 * r->experts + r->groups) * sizeof(float);
  const size_t small = tokens * (per_warp + r->top * sizeof(int));
  if (tokens <= kRouteSmallTokens && small <= 40 * 1024) {
    const int need = (int)tokens * 32 > r->experts ? (int)tokens * 32 : r->experts, threads = (need + 31) / 32 * 32;
    return launch_overlapped(moe_route_small_kernel, dim3(1), dim3((unsigned)threads), small, st, logits, *r, *plan, (int)tokens);
  }
  if (cudaMemsetAsync(plan->counters, 0, (size_t)r->experts * sizeof(int32_t), st) != cudaSuccess) { cudaGetLastError(); return NQB200_ERR_LAUNCH; }
  const size_t smem = kRouteWarps * per_warp;
  if (smem > 40 * 1024 && cudaFuncSetAttribute(moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return NQB200_ERR_LAUNCH;
  }
  int rc = launch_overlapped(moe_route_kernel, dim3((unsigned)((tokens + kRouteWarps - 1) / kRouteWarps)), dim3(kRouteWarps * 32), smem, st, logits, *r, *plan,
                             (int)tokens);
  if (rc == NQB200_OK) rc = launch_overlapped(moe_scan_kernel, dim3(1), dim3((unsigned)((r->experts + 31) / 32 * 32)), 0, st, *plan, r->experts);
  const int pairs = (int)tokens * r->top, per = 256 * kScatterPairs;
  if (rc == NQB200_OK) rc = launch_overlapped(moe_scatter_kernel, dim3((unsigned)((pairs + per - 1) / per)), dim3(256), 0, st, *plan, r->experts, pairs);
  return rc;
}
