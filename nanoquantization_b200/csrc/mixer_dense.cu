// Skinny dense linears (up to 16 tokens, bf16 weights [N, K] row-major) of decode steps, with the step that follows
// them inside: residual add into the float stream, clamped GLU, minGRU update.
//
// A CTA owns 16 outputs; its 8 warps split K in interleaved blocks of 32.  Weights go from global memory to the
// operand registers of mma.m16n8k16 directly: lane (g, t) loads 16 bytes (8 consecutive k) of rows g and g + 8, and
// the same 8 k of token g; which k a lane's registers stand for does not matter to a dot product as long as both
// operands agree.  The first batch of weights is requested before the kernel waits for the one ahead of it.
#include "mixers.cuh"

namespace nqb200 {

enum DenseMode { kPlain = 0, kFloat = 1, kResidual = 2, kGlu = 3, kMinGru = 4, kTable = 5 };

struct DenseArgs {
  const bf16* x; const bf16* w; void* out;
  int M, N, K;            // N: rows of one group (outputs)
  float beta;             // residual
  float limit;            // GLU
  const float* z_bias; const float* x_bias; float* state; const int32_t* slot; const int32_t* pos0;  // minGRU
  const int64_t* ids; const bf16* table; int64_t table_stride;   // token table (its first column added)
};

__device__ __forceinline__ uint4 ld_weight(const bf16* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.L2::256B.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

__device__ __forceinline__ void mma16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int MODE, int MT>
__global__ void __launch_bounds__(256) dense_decode_kernel(const DenseArgs p) {
  constexpr int NG = MODE == kMinGru ? 3 : MODE == kGlu ? 2 : 1;      // row groups that meet in one output
  constexpr int U = MODE == kMinGru ? 2 : MODE == kGlu ? 4 : 8;       // k-blocks in flight per warp
  __shared__ float part[8][NG][MT * 8][16 + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int n0 = blockIdx.x * 16, blocks = (p.K + 31) / 32;
  const bf16* wrow[NG][2];
#pragma unroll
  for (int q = 0; q < NG; ++q)
#pragma unroll
    for (int r = 0; r < 2; ++r) wrow[q][r] = p.w + ((size_t)q * p.N + min(n0 + g + 8 * r, p.N - 1)) * p.K + t * 8;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  uint4 wv[U][NG][2];
  auto fetch = [&](int kb0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int kb = kb0 + u * 8;
      const bool ok = kb < blocks && kb * 32 + t * 8 < p.K;   // K is a multiple of 8
#pragma unroll
      for (int q = 0; q < NG; ++q)
#pragma unroll
        for (int r = 0; r < 2; ++r) wv[u][q][r] = ok ? ld_weight(wrow[q][r] + kb * 32) : zero;
    }
  };
  float acc[NG][MT][4] = {};
  fetch(warp);
  grid_launch_dependents();
  grid_dependency_wait();
  for (int kb0 = warp; kb0 < blocks; kb0 += 8 * U) {
    uint4 xv[U][MT];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = (kb0 + u * 8) * 32 + t * 8;
#pragma unroll
      for (int m = 0; m < MT; ++m)
        xv[u][m] = (k < p.K && m * 8 + g < p.M) ? *reinterpret_cast<const uint4*>(p.x + (size_t)(m * 8 + g) * p.K + k) : zero;
    }
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int q = 0; q < NG; ++q)
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          const uint4 a = wv[u][q][0], b = wv[u][q][1], x = xv[u][m];
          mma16816(acc[q][m], a.x, b.x, a.y, b.y, x.x, x.y);
          mma16816(acc[q][m], a.z, b.z, a.w, b.w, x.z, x.w);
        }
    if (kb0 + 8 * U < blocks) fetch(kb0 + 8 * U);
  }
#pragma unroll
  for (int q = 0; q < NG; ++q)
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int e = 0; e < 4; ++e) part[warp][q][m * 8 + t * 2 + (e & 1)][g + 8 * (e >> 1)] = acc[q][m][e];
  __syncthreads();
  const int row = threadIdx.x % 16, tok = threadIdx.x / 16, n = n0 + row;
  if (tok >= MT * 8 || tok >= p.M || n >= p.N) return;
  float v[NG];
#pragma unroll
  for (int q = 0; q < NG; ++q) {
    v[q] = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) v[q] += part[w][q][tok][row];
  }
  const size_t at = (size_t)tok * p.N + n;
  if (MODE == kPlain) {
    reinterpret_cast<bf16*>(p.out)[at] = __float2bfloat16_rn(v[0]);
  } else if (MODE == kFloat) {
    reinterpret_cast<float*>(p.out)[at] = v[0];
  } else if (MODE == kResidual) {
    float* o = reinterpret_cast<float*>(p.out) + at;
    *o = p.beta * *o + v[0];
  } else if (MODE == kTable) {
    reinterpret_cast<bf16*>(p.out)[at] = __float2bfloat16_rn(gelu_tanh_f(v[0]) * to_f(p.table[(size_t)p.ids[tok] * p.table_stride + n]));
  } else if (MODE == kGlu) {
    const float gt = fminf(v[0], p.limit), up = fminf(fmaxf(v[NG - 1], -p.limit), p.limit);
    reinterpret_cast<bf16*>(p.out)[at] = __float2bfloat16_rn(gt * sigmoid_f(1.702f * gt) * (up + 1.f));
  } else {
    float* st = p.state + (size_t)p.slot[tok] * p.N + n;
    const float z = sigmoid_f(v[0] + p.z_bias[n]), u = v[1 % NG] + p.x_bias[n], gt = v[NG - 1];
    const float cand = u >= 0.f ? u + 0.5f : sigmoid_f(u);
    const float S = (1.f - z) * (p.pos0[tok] != 0 ? *st : 0.f) + z * cand;
    *st = S;
    reinterpret_cast<bf16*>(p.out)[at] = __float2bfloat16_rn(S * (gt * sigmoid_f(gt)));
  }
}

template <int MODE>
static int launch_dense(const DenseArgs& p, cudaStream_t st) {
  if (p.M < 0 || p.M > 16 || p.N <= 0 || p.K <= 0 || p.K % 8 != 0) return NQB200_ERR_BAD_SHAPE;
  if (p.M == 0) return NQB200_OK;
  if (!p.x || !p.w || !p.out) return NQB200_ERR_NULL_POINTER;
  if (!aligned16(p.x) || !aligned16(p.w)) return NQB200_ERR_MISALIGNED;
  const dim3 grid((unsigned)((p.N + 15) / 16)), block(256);
  return p.M <= 8 ? launch_overlapped(dense_decode_kernel<MODE, 1>, grid, block, 0, st, p) : launch_overlapped(dense_decode_kernel<MODE, 2>, grid, block, 0, st, p);
}

}  // namespace nqb200

using namespace nqb200;

static bool dense_sizes(int64_t M, int64_t N, int64_t K) { return M >= 0 && M <= 16 && N > 0 && K > 0 && N <= (1 << 28) && K <= (1 << 28); }

extern "C" int nqb200_dense_decode(const void* x, const void* w, void* out, int64_t M, int64_t N, int64_t K, int mode, float beta, void* stream) {
  if (!dense_sizes(M, N, K)) return NQB200_ERR_BAD_SHAPE;
  DenseArgs p = {};
  p.x = (const bf16*)x; p.w = (const bf16*)w; p.out = out; p.M = (int)M; p.N = (int)N; p.K = (int)K; p.beta = beta;
  cudaStream_t st = (cudaStream_t)stream;
  if (mode == NQB200_DENSE_BF16) return launch_dense<kPlain>(p, st);
  if (mode == NQB200_DENSE_F32) return launch_dense<kFloat>(p, st);
  if (mode == NQB200_DENSE_RESIDUAL) return launch_dense<kResidual>(p, st);
  return NQB200_ERR_BAD_DTYPE;
}

extern "C" int nqb200_dense_decode_gelu_table(const void* x, const void* w, const int64_t* ids, const void* table, int64_t table_stride,
                                              int64_t column, void* out, int64_t M, int64_t dim, int64_t K, void* stream) {
  if (!dense_sizes(M, dim, K) || column < 0 || table_stride < column + dim) return NQB200_ERR_BAD_SHAPE;
  if (M > 0 && (!ids || !table)) return NQB200_ERR_NULL_POINTER;
  DenseArgs p = {};
  p.x = (const bf16*)x; p.w = (const bf16*)w; p.out = out; p.M = (int)M; p.N = (int)dim; p.K = (int)K;
  p.ids = ids; p.table = (const bf16*)table + column; p.table_stride = table_stride;
  return launch_dense<kTable>(p, (cudaStream_t)stream);
}

extern "C" int nqb200_dense_decode_glu(const void* x, const void* w, void* out, int64_t M, int64_t ff, int64_t K, float limit, void* stream) {
  if (!dense_sizes(M, ff, K)) return NQB200_ERR_BAD_SHAPE;
  DenseArgs p = {};
  p.x = (const bf16*)x; p.w = (const bf16*)w; p.out = out; p.M = (int)M; p.N = (int)ff; p.K = (int)K; p.limit = limit;
  return launch_dense<kGlu>(p, (cudaStream_t)stream);
}

extern "C" int nqb200_dense_decode_mingru(const void* x, const void* w, const float* z_bias, const float* x_bias, float* state, void* out,
                                          int64_t width, int64_t K, const nqb200_batch* b, void* stream) {
  const int s = check_batch(b, false);
  if (s != NQB200_OK) return s;
  if (!dense_sizes(b->tokens, width, K) || b->max_len > 1 || b->tokens != b->batch) return NQB200_ERR_BAD_SHAPE;
  if (b->tokens > 0 && (!z_bias || !x_bias || !state)) return NQB200_ERR_NULL_POINTER;
  DenseArgs p = {};
  p.x = (const bf16*)x; p.w = (const bf16*)w; p.out = out; p.M = b->tokens; p.N = (int)width; p.K = (int)K;
  p.z_bias = z_bias; p.x_bias = x_bias; p.state = state; p.slot = b->slot; p.pos0 = b->pos0;
  return launch_dense<kMinGru>(p, (cudaStream_t)stream);
}
