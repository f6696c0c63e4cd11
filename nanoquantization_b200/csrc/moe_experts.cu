// The experts' linears over pairs sorted by expert: a kernel for any size and type, and one for decode steps that streams
// the weights of every expert that has tokens once.  The tcgen05 kernel for larger steps is in moe_umma.cu.
#include "moe.cuh"

namespace nqb200 {

struct MoeDevice {
  const void* x; const void* w; void* out;
  int kind, N, K, top;
  const int32_t* offsets; const int32_t* order; const int32_t* active; const float* weight;
};

template <typename O>
__device__ __forceinline__ void moe_store(const MoeDevice& p, int i, int n, float v) {   // value n of the i-th pair in the plan's order
  if (p.kind == NQB200_MOE_UP) {
    reinterpret_cast<O*>(p.out)[(size_t)i * p.N + n] = from_f<O>(gelu_erf_f(v));
  } else {
    const int pair = p.order[i];
    reinterpret_cast<O*>(p.out)[(size_t)pair * p.N + n] = from_f<O>(p.weight[pair] * v);
  }
}

constexpr int kSimpleTok = 32, kSimpleOut = 64, kSimpleK = 32;
template <typename T, typename O>
__global__ void __launch_bounds__(256) moe_simple_kernel(const MoeDevice p) {
  __shared__ float xs[kSimpleTok][kSimpleK + 1], ws[kSimpleOut][kSimpleK + 1];
  grid_launch_dependents();
  grid_dependency_wait();
  const int e = blockIdx.z, lo = p.offsets[e] + blockIdx.y * kSimpleTok, cnt = min(kSimpleTok, p.offsets[e + 1] - lo), n0 = blockIdx.x * kSimpleOut;
  if (cnt <= 0) return;
  const int tid = threadIdx.x, tx = tid % 16, ty = tid / 16;   // outputs tx + 16 j, tokens ty + 16 i
  float acc[2][4] = {};
  const T* w = reinterpret_cast<const T*>(p.w) + (size_t)e * p.N * p.K;
  for (int k0 = 0; k0 < p.K; k0 += kSimpleK) {
    for (int q = tid; q < kSimpleTok * kSimpleK; q += 256) {
      const int i = q / kSimpleK, k = k0 + q % kSimpleK;
      const int row = i < cnt ? (p.kind == NQB200_MOE_UP ? p.order[lo + i] / p.top : lo + i) : 0;
      xs[i][q % kSimpleK] = (i < cnt && k < p.K) ? to_f(reinterpret_cast<const T*>(p.x)[(size_t)row * p.K + k]) : 0.f;
    }
    for (int q = tid; q < kSimpleOut * kSimpleK; q += 256) {
      const int j = q / kSimpleK, k = k0 + q % kSimpleK;
      ws[j][q % kSimpleK] = (n0 + j < p.N && k < p.K) ? to_f(w[(size_t)(n0 + j) * p.K + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < kSimpleK; ++k)
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += xs[ty + 16 * i][k] * ws[tx + 16 * j][k];
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (ty + 16 * i < cnt && n0 + tx + 16 * j < p.N) moe_store<O>(p, lo + ty + 16 * i, n0 + tx + 16 * j, acc[i][j]);
}

// Decode steps (bf16, at most 16 tokens): a CTA owns 16 outputs of one expert, its 8 warps split K in interleaved blocks of
// 32, and weights go from global memory to the operand registers of mma.m16n8k16 directly (as the dense decode linears).
__device__ __forceinline__ uint4 moe_ld_weight(const bf16* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.L2::256B.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
__device__ __forceinline__ void moe_mma(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <typename O, int MT>
__global__ void __launch_bounds__(256) moe_decode_kernel(const MoeDevice p) {
  constexpr int U = 8;      // k-blocks in flight per warp
  __shared__ float part[8][MT * 8][16 + 1];
  grid_launch_dependents();
  grid_dependency_wait();
  if ((int)blockIdx.y >= p.active[0]) return;
  const int e = p.active[1 + blockIdx.y], lo = p.offsets[e], cnt = min(p.offsets[e + 1] - lo, MT * 8);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int n0 = blockIdx.x * 16, blocks = (p.K + 31) / 32;
  const bf16* w = reinterpret_cast<const bf16*>(p.w) + (size_t)e * p.N * p.K + t * 8;
  const bf16* w0 = w + (size_t)min(n0 + g, p.N - 1) * p.K;
  const bf16* w1 = w + (size_t)min(n0 + g + 8, p.N - 1) * p.K;
  const bf16* xr[MT];
#pragma unroll
  for (int m = 0; m < MT; ++m) {
    const int i = min(m * 8 + g, cnt - 1);
    xr[m] = reinterpret_cast<const bf16*>(p.x) + (size_t)(p.kind == NQB200_MOE_UP ? p.order[lo + i] / p.top : lo + i) * p.K + t * 8;
  }
  const uint4 zero = make_uint4(0, 0, 0, 0);
  float acc[MT][4] = {};
  for (int kb0 = warp; kb0 < blocks; kb0 += 8 * U) {
    uint4 wv[U][2], xv[U][MT];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = (kb0 + u * 8) * 32;
      const bool ok = k + t * 8 < p.K;   // K is a multiple of 8
      wv[u][0] = ok ? moe_ld_weight(w0 + k) : zero;
      wv[u][1] = ok ? moe_ld_weight(w1 + k) : zero;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = (kb0 + u * 8) * 32;
#pragma unroll
      for (int m = 0; m < MT; ++m) xv[u][m] = (k + t * 8 < p.K && m * 8 + g < cnt) ? *reinterpret_cast<const uint4*>(xr[m] + k) : zero;
    }
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const uint4 a = wv[u][0], b = wv[u][1], x = xv[u][m];
        moe_mma(acc[m], a.x, b.x, a.y, b.y, x.x, x.y);
        moe_mma(acc[m], a.z, b.z, a.w, b.w, x.z, x.w);
      }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int c = 0; c < 4; ++c) part[warp][m * 8 + t * 2 + (c & 1)][g + 8 * (c >> 1)] = acc[m][c];
  __syncthreads();
  const int row = threadIdx.x % 16, tok = threadIdx.x / 16, n = n0 + row;
  if (tok >= cnt || n >= p.N) return;
  float v = 0.f;
#pragma unroll
  for (int q = 0; q < 8; ++q) v += part[q][tok][row];
  moe_store<O>(p, lo + tok, n, v);
}

static MoeDevice device_args(const MoeArgs& a) {
  MoeDevice p = {};
  p.x = a.x; p.w = a.w; p.out = a.out; p.kind = a.kind; p.N = a.N; p.K = a.K; p.top = a.top;
  p.offsets = a.plan.offsets; p.order = a.plan.order; p.active = a.plan.active; p.weight = a.plan.weight;
  return p;
}

bool moe_decode_supports(int64_t tokens, int64_t N, int64_t K) { return tokens <= kMoeDecodeTokens && K % 8 == 0 && N > 0; }
int moe_decode(const MoeArgs& a) {
  const MoeDevice p = device_args(a);
  const int most = a.tokens * a.top < a.experts ? a.tokens * a.top : a.experts;
  const dim3 grid((unsigned)((a.N + 15) / 16), (unsigned)most), block(256);
  if (a.out_dtype == NQB200_F32)
    return a.tokens <= 8 ? launch_overlapped(moe_decode_kernel<float, 1>, grid, block, 0, a.stream, p) : launch_overlapped(moe_decode_kernel<float, 2>, grid, block, 0, a.stream, p);
  return a.tokens <= 8 ? launch_overlapped(moe_decode_kernel<bf16, 1>, grid, block, 0, a.stream, p) : launch_overlapped(moe_decode_kernel<bf16, 2>, grid, block, 0, a.stream, p);
}

static int moe_simple(const MoeArgs& a) {
  const MoeDevice p = device_args(a);
  const int64_t ty = (a.tokens + kSimpleTok - 1) / kSimpleTok;
  if (ty > 65535) return NQB200_ERR_TOO_LARGE;
  const dim3 grid((unsigned)((a.N + kSimpleOut - 1) / kSimpleOut), (unsigned)ty, (unsigned)a.experts), block(256);
  if (a.dtype == NQB200_F32) return launch_overlapped(moe_simple_kernel<float, float>, grid, block, 0, a.stream, p);
  if (a.out_dtype == NQB200_F32) return launch_overlapped(moe_simple_kernel<bf16, float>, grid, block, 0, a.stream, p);
  return launch_overlapped(moe_simple_kernel<bf16, bf16>, grid, block, 0, a.stream, p);
}

}  // namespace nqb200

using namespace nqb200;

extern "C" const char* nqb200_moe_linear_kernel(int64_t tokens, int64_t N, int64_t K, int64_t top, int dtype) {
  if (dtype == NQB200_BF16 && moe_decode_supports(tokens, N, K)) return "decode";
  if (dtype == NQB200_BF16 && moe_umma_supports(tokens, N, K, top)) return "tcgen05";
  return "simple";
}

extern "C" int nqb200_moe_linear(const void* x, const void* w, void* out, int kind, int64_t tokens, int64_t N, int64_t K, const nqb200_router* r,
                                 const nqb200_moe_plan* plan, int dtype, int out_dtype, int* status, void* stream) {
  if (!r || !plan) return NQB200_ERR_NULL_POINTER;
  if (tokens < 0 || N <= 0 || K <= 0 || r->experts <= 0 || r->experts > 65535 || r->top <= 0 || tokens * r->top > INT32_MAX || N > (1 << 24) || K > (1 << 24) ||
      (kind != NQB200_MOE_UP && kind != NQB200_MOE_DOWN))
    return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype) || !mixer_dtype(out_dtype) || (dtype == NQB200_F32 && out_dtype != NQB200_F32) || (kind == NQB200_MOE_UP && out_dtype != dtype))
    return NQB200_ERR_BAD_DTYPE;
  if (tokens == 0) return NQB200_OK;
  if (!x || !w || !out || !plan->offsets || !plan->order || !plan->active || !plan->weight) return NQB200_ERR_NULL_POINTER;
  if (!aligned16(x) || !aligned16(w) || !aligned16(out)) return NQB200_ERR_MISALIGNED;
  MoeArgs a = {};
  a.x = x; a.w = w; a.out = out; a.kind = kind; a.tokens = (int)tokens; a.N = (int)N; a.K = (int)K; a.experts = r->experts; a.top = r->top;
  a.plan = *plan; a.dtype = dtype; a.out_dtype = out_dtype; a.status = status; a.stream = (cudaStream_t)stream;
  if (dtype == NQB200_BF16 && moe_decode_supports(tokens, N, K)) return moe_decode(a);
  if (dtype == NQB200_BF16 && out_dtype == NQB200_BF16 && a.experts <= 1024 && a.experts * N >= 128 && moe_umma_supports(tokens, N, K, r->top)) return moe_umma(a);
  return moe_simple(a);
}
