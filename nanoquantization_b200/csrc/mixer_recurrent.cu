// Recurrences over tokens with a float state per sequence: retention (a matrix per head with a fixed decay) and
// minGRU (an element-wise gated scan).  Kernels here take any sizes and both element types.
#include "mixers.cuh"

namespace nqb200 {

constexpr int kRetCols = 32, kRetGroups = 8, kRetTokens = 16;

// One CTA per (32 value columns, head, sequence), tokens in order.  Thread (group, column) keeps rows
// group, group + 8, ... of its column of S in registers.
template <typename T, int DPT>
__global__ void __launch_bounds__(kRetCols* kRetGroups) retention_simple_kernel(const T* __restrict__ proj, int64_t stride, int q_off, int k_off,
                                                                                int v_off, const float* __restrict__ decay,
                                                                                const float* __restrict__ log_decay, float* state,
                                                                                float* __restrict__ o, int heads, int dim, int vdim,
                                                                                const nqb200_batch bt) {
  extern __shared__ float sm[];
  float* qs = sm;                               // [tokens][dim]
  float* ks = qs + kRetTokens * dim;            // [tokens][dim], scaled
  float* vs = ks + kRetTokens * dim;            // [tokens][cols]
  float* part = vs + kRetTokens * kRetCols;     // [tokens][groups][cols]
  float* ds = part + kRetTokens * kRetGroups * kRetCols;   // [tokens][dim] decays, where every channel has its own
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.z, h = blockIdx.y, col = threadIdx.x % kRetCols, grp = threadIdx.x / kRetCols, tid = threadIdx.x;
  const int c = blockIdx.x * kRetCols + col, t0 = bt.cu[b], n = bt.cu[b + 1] - t0;
  if (n <= 0) return;
  float* st = state + ((size_t)bt.slot[b] * heads + h) * dim * vdim;
  const bool live = c < vdim, fresh = bt.pos0[b] == 0;
  const float d = log_decay ? 0.f : decay[h], kscale = 1.f / sqrtf((float)dim);
  float S[DPT];
#pragma unroll
  for (int r = 0; r < DPT; ++r) {
    const int row = r * kRetGroups + grp;
    S[r] = (live && !fresh && row < dim) ? st[(size_t)row * vdim + c] : 0.f;
  }
  for (int base = 0; base < n; base += kRetTokens) {
    const int cnt = min(kRetTokens, n - base);
    __syncthreads();
    for (int e = tid; e < cnt * dim; e += blockDim.x) {
      const int i = e / dim, r = e - i * dim;
      const T* row = proj + (size_t)(t0 + base + i) * stride + (size_t)h * dim + r;
      qs[e] = to_f(row[q_off]);
      ks[e] = to_f(row[k_off]) * kscale;
      if (log_decay) ds[e] = expf(log_decay[((size_t)(t0 + base + i) * heads + h) * dim + r]);
    }
    for (int e = tid; e < cnt * kRetCols; e += blockDim.x) {
      const int i = e / kRetCols, cc = blockIdx.x * kRetCols + e % kRetCols;
      vs[e] = cc < vdim ? to_f(proj[(size_t)(t0 + base + i) * stride + v_off + (size_t)h * vdim + cc]) : 0.f;
    }
    __syncthreads();
    for (int i = 0; i < cnt; ++i) {
      const float v = vs[i * kRetCols + col];
      float acc = 0.f;
#pragma unroll
      for (int r = 0; r < DPT; ++r) {
        const int row = r * kRetGroups + grp;
        if (row < dim) {
          S[r] = (log_decay ? ds[i * dim + row] : d) * S[r] + ks[i * dim + row] * v;
          acc += S[r] * qs[i * dim + row];
        }
      }
      part[(i * kRetGroups + grp) * kRetCols + col] = acc;
    }
    __syncthreads();
    for (int e = tid; e < cnt * kRetCols; e += blockDim.x) {
      const int i = e / kRetCols, cc = blockIdx.x * kRetCols + e % kRetCols;
      if (cc >= vdim) continue;
      float acc = 0.f;
#pragma unroll
      for (int g = 0; g < kRetGroups; ++g) acc += part[(i * kRetGroups + g) * kRetCols + e % kRetCols];
      o[((size_t)(t0 + base + i) * heads + h) * vdim + cc] = acc;
    }
  }
  if (live) {
#pragma unroll
    for (int r = 0; r < DPT; ++r) {
      const int row = r * kRetGroups + grp;
      if (row < dim) st[(size_t)row * vdim + c] = S[r];
    }
  }
}

// One warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* __restrict__ o, const T* __restrict__ gate, int64_t gate_stride,
                                                             const float* __restrict__ weight, T* __restrict__ out, int64_t out_stride, int64_t pairs, int heads, int vdim,
                                                             float eps, float out_scale) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int64_t w = blockIdx.x * (int64_t)(blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= pairs) return;
  const int64_t t = w / heads;
  const int h = (int)(w - t * heads), lane = threadIdx.x & 31;
  const float* row = o + w * vdim;
  float ss = 0.f;
  for (int c = lane; c < vdim; c += 32) ss += row[c] * row[c];
  const float inv = out_scale / sqrtf(warp_sum(ss) / (float)vdim + eps);
  for (int c = lane; c < vdim; c += 32) {
    const float g = to_f(gate[t * gate_stride + (int64_t)h * vdim + c]);
    out[t * out_stride + (int64_t)h * vdim + c] = from_f<T>(row[c] * inv * (weight ? weight[c] : 1.f) * (g * sigmoid_f(g)));
  }
}

// A thread per channel and 16 tokens: log of the decays, from the gate's low-rank projection.
constexpr int kDecayTokens = 16;
template <typename T>
__global__ void __launch_bounds__(256) gla_log_decay_kernel(const T* __restrict__ low, int64_t low_stride, const T* __restrict__ a2,
                                                            const float* __restrict__ bias, float* __restrict__ out, int64_t tokens, int channels,
                                                            int rank, float inv_tau) {
  extern __shared__ float low_s[];   // [kDecayTokens][rank]
  grid_launch_dependents();
  grid_dependency_wait();
  const int64_t t0 = (int64_t)blockIdx.y * kDecayTokens;
  const int cnt = (int)min((int64_t)kDecayTokens, tokens - t0);
  for (int e = threadIdx.x; e < cnt * rank; e += 256) low_s[e] = to_f(low[(t0 + e / rank) * low_stride + e % rank]);
  __syncthreads();
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= channels) return;
  float z[kDecayTokens];
  const float b = bias[c];
#pragma unroll
  for (int i = 0; i < kDecayTokens; ++i) z[i] = 0.f;
  for (int r = 0; r < rank; ++r) {
    const float w = to_f(a2[(size_t)c * rank + r]);
#pragma unroll
    for (int i = 0; i < kDecayTokens; ++i) z[i] += w * (i < cnt ? low_s[i * rank + r] : 0.f);
  }
#pragma unroll
  for (int i = 0; i < kDecayTokens; ++i)
    if (i < cnt) out[(t0 + i) * channels + c] = log_sigmoid_f(z[i] + b) * inv_tau;
}

constexpr int kGruSegs = 32, kGruCols = 32, kGruLen = 4;  // 128 tokens per pass

// One CTA per (32 channels, sequence).  Thread (segment, channel) folds its 4 tokens into S -> A S + B, a warp per
// channel scans the 32 segments, and the thread replays its tokens from the state at its segment's start.
template <typename T>
__global__ void __launch_bounds__(kGruSegs* kGruCols) mingru_kernel(const T* __restrict__ proj, int64_t stride, int z_off, int x_off, int g_off,
                                                                    const float* __restrict__ z_bias, const float* __restrict__ x_bias,
                                                                    float* state, T* __restrict__ out, int width, const nqb200_batch bt) {
  __shared__ float As[kGruSegs][kGruCols + 1], Bs[kGruSegs][kGruCols + 1], carry[kGruCols];
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.y, col = threadIdx.x % kGruCols, seg = threadIdx.x / kGruCols, c = blockIdx.x * kGruCols + col;
  const int t0 = bt.cu[b], n = bt.cu[b + 1] - t0;
  if (n <= 0) return;
  const bool live = c < width;
  float* st = state + (size_t)bt.slot[b] * width;
  const float zb = live ? z_bias[c] : 0.f, xb = live ? x_bias[c] : 0.f;
  if (seg == 0) carry[col] = live && bt.pos0[b] != 0 ? st[c] : 0.f;
  for (int base = 0; base < n; base += kGruSegs * kGruLen) {
    float a[kGruLen], v[kGruLen], A = 1.f, B = 0.f;
#pragma unroll
    for (int i = 0; i < kGruLen; ++i) {
      const int tok = base + seg * kGruLen + i;
      a[i] = 1.f; v[i] = 0.f;
      if (live && tok < n) {
        const T* row = proj + (size_t)(t0 + tok) * stride;
        const float z = sigmoid_f(to_f(row[z_off + c]) + zb), u = to_f(row[x_off + c]) + xb;
        a[i] = 1.f - z;
        v[i] = z * (u >= 0.f ? u + 0.5f : sigmoid_f(u));
      }
      A *= a[i];
      B = a[i] * B + v[i];
    }
    As[seg][col] = A;
    Bs[seg][col] = B;
    __syncthreads();
    {
      // warp `seg` scans channel `seg`; its lanes are the segments
      const int ch = seg, lane = col;
      float sa = As[lane][ch], sb = Bs[lane][ch];
#pragma unroll
      for (int off = 1; off < 32; off <<= 1) {
        const float pa = __shfl_up_sync(0xFFFFFFFFu, sa, off), pb = __shfl_up_sync(0xFFFFFFFFu, sb, off);
        if (lane >= off) { sb = sa * pb + sb; sa = sa * pa; }
      }
      const float s0 = carry[ch], end = sa * s0 + sb;
      float begin = __shfl_up_sync(0xFFFFFFFFu, end, 1);
      if (lane == 0) begin = s0;
      Bs[lane][ch] = begin;
      __syncwarp();
      if (lane == 31) carry[ch] = end;
    }
    __syncthreads();
    float S = Bs[seg][col];
#pragma unroll
    for (int i = 0; i < kGruLen; ++i) {
      const int tok = base + seg * kGruLen + i;
      S = a[i] * S + v[i];
      if (live && tok < n) {
        const float g = to_f(proj[(size_t)(t0 + tok) * stride + g_off + c]);
        out[(size_t)(t0 + tok) * width + c] = from_f<T>(S * (g * sigmoid_f(g)));
      }
    }
    __syncthreads();
  }
  if (seg == 0 && live) st[c] = carry[col];
}

// Two channels per thread (even widths): a CTA takes 64 channels x 128 tokens, a warp 16 of the tokens, so that the
// chunks of a prompt run side by side.  A first launch folds each chunk into S -> A S + B, a second walks over the folds
// and leaves every chunk's starting state in its fold's place, and the third scans its 8 warps' folds and replays the
// tokens.
constexpr int kGruChunk = 128, kGruWarpTokens = 16;

__device__ __forceinline__ float2 ld_pair(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ld_pair(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void st_pair(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void st_pair(bf16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }
template <typename T> __device__ __forceinline__ float gate_sigmoid(float v) { return sigmoid_f(v); }
template <> __device__ __forceinline__ float gate_sigmoid<bf16>(float v) { return sigmoid_fast(v); }

struct GruArgs {
  int64_t stride;
  int z_off, x_off, g_off, width;
  const float* z_bias; const float* x_bias;
  float* state; float2* folds;   // folds [chunk id][width / 2]: A of both channels, then B of both
  nqb200_batch bt;
};
__device__ __forceinline__ size_t gru_chunk_id(const nqb200_batch& bt, int b, int c) { return (size_t)(bt.cu[b] / kGruChunk + b + c); }

template <typename T, bool FOLD>
__global__ void __launch_bounds__(256) mingru_chunk_kernel(const T* __restrict__ proj, T* __restrict__ out, const GruArgs p) {
  __shared__ float2 As[8][32], Bs[8][32];
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.z, chunk = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t0 = p.bt.cu[b], n = p.bt.cu[b + 1] - t0, first = chunk * kGruChunk, c = blockIdx.x * 64 + lane * 2;
  if (first >= n) return;
  const bool live = c < p.width, fresh = p.bt.pos0[b] == 0;
  const int tok0 = first + warp * kGruWarpTokens, cnt = max(0, min(kGruWarpTokens, n - tok0));
  float* own = p.state + (size_t)p.bt.slot[b] * p.width + c;
  float2 a[kGruWarpTokens], v[kGruWarpTokens], A = make_float2(1.f, 1.f), B = make_float2(0.f, 0.f);
  const float2 zb = live ? ld_pair(p.z_bias + c) : B, xb = live ? ld_pair(p.x_bias + c) : B;
  // every load is made, from a place that exists (what does not count is masked below), so that all are under way at once
  const T* base = proj + (live ? c : 0);
#pragma unroll
  for (int i = 0; i < kGruWarpTokens; ++i) {
    const T* row = base + (size_t)(t0 + min(tok0 + i, n - 1)) * p.stride;
    a[i] = ld_pair(row + p.z_off);
    v[i] = ld_pair(row + p.x_off);
  }
#pragma unroll
  for (int i = 0; i < kGruWarpTokens; ++i) {
    const float zx = gate_sigmoid<T>(a[i].x + zb.x), zy = gate_sigmoid<T>(a[i].y + zb.y), ux = v[i].x + xb.x, uy = v[i].y + xb.y;
    const bool ok = i < cnt;
    a[i] = ok ? make_float2(1.f - zx, 1.f - zy) : make_float2(1.f, 1.f);
    v[i] = ok ? make_float2(zx * (ux >= 0.f ? ux + 0.5f : gate_sigmoid<T>(ux)), zy * (uy >= 0.f ? uy + 0.5f : gate_sigmoid<T>(uy))) : make_float2(0.f, 0.f);
    A.x *= a[i].x; A.y *= a[i].y;
    B.x = a[i].x * B.x + v[i].x; B.y = a[i].y * B.y + v[i].y;
  }
  As[warp][lane] = A;
  Bs[warp][lane] = B;
  float2 S = make_float2(0.f, 0.f);   // FOLD: the fold's own B; else the state at the chunk's start
  if (!FOLD && live) {
    if (n > kGruChunk) S = p.folds[2 * (gru_chunk_id(p.bt, b, chunk) * (p.width / 2) + c / 2)];   // where the scan left it
    else if (!fresh) S = ld_pair(own);
  }
  __syncthreads();
  if constexpr (FOLD) {
    if (warp == 0 && live) {
      float2 FA = make_float2(1.f, 1.f), FB = make_float2(0.f, 0.f);
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        const float2 wa = As[w][lane], wb = Bs[w][lane];
        FA.x *= wa.x; FA.y *= wa.y;
        FB.x = wa.x * FB.x + wb.x; FB.y = wa.y * FB.y + wb.y;
      }
      *reinterpret_cast<float4*>(p.folds + 2 * (gru_chunk_id(p.bt, b, chunk) * (p.width / 2) + c / 2)) = make_float4(FA.x, FA.y, FB.x, FB.y);
    }
  } else {
    for (int w = 0; w < warp; ++w) {
      const float2 wa = As[w][lane], wb = Bs[w][lane];
      S.x = wa.x * S.x + wb.x; S.y = wa.y * S.y + wb.y;
    }
    T* orow = out + (size_t)(t0 + tok0) * p.width + c;
    float2 gate[kGruWarpTokens];
#pragma unroll
    for (int i = 0; i < kGruWarpTokens; ++i) gate[i] = ld_pair(base + (size_t)(t0 + min(tok0 + i, n - 1)) * p.stride + p.g_off);
#pragma unroll
    for (int i = 0; i < kGruWarpTokens; ++i) {
      S.x = a[i].x * S.x + v[i].x; S.y = a[i].y * S.y + v[i].y;
      if (live && i < cnt) {
        const float2 g = gate[i];
        st_pair(orow + (size_t)i * p.width, make_float2(S.x * (g.x * gate_sigmoid<T>(g.x)), S.y * (g.y * gate_sigmoid<T>(g.y))));
      }
    }
    // every warp has read the state (of a sequence with one chunk) before the last one replaces it
    __syncthreads();
    if (live && warp == 7 && first + kGruChunk >= n) st_pair(own, S);
  }
}

__global__ void __launch_bounds__(64) mingru_scan_kernel(const GruArgs p) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.y, pair = blockIdx.x * 64 + threadIdx.x, n = p.bt.cu[b + 1] - p.bt.cu[b];
  if (pair * 2 >= p.width || n <= kGruChunk) return;
  const int chunks = (n + kGruChunk - 1) / kGruChunk;
  float2 S = p.bt.pos0[b] == 0 ? make_float2(0.f, 0.f) : ld_pair(p.state + (size_t)p.bt.slot[b] * p.width + pair * 2);
  float2* f = p.folds + 2 * (gru_chunk_id(p.bt, b, 0) * (p.width / 2) + pair);
  for (int c0 = 0; c0 < chunks; c0 += 16) {
    float4 ab[16];
#pragma unroll
    for (int k = 0; k < 16; ++k) ab[k] = *reinterpret_cast<const float4*>(f + (size_t)min(c0 + k, chunks - 1) * p.width);
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      if (c0 + k >= chunks) break;
      f[(size_t)(c0 + k) * p.width] = S;
      S.x = ab[k].x * S.x + ab[k].z;
      S.y = ab[k].y * S.y + ab[k].w;
    }
  }
}

}  // namespace nqb200

using namespace nqb200;

template <typename T>
static int mingru_chunked(const void* proj, void* out, const GruArgs& p, cudaStream_t st) {
  const dim3 grid((unsigned)((p.width + 63) / 64), (unsigned)((p.bt.max_len + kGruChunk - 1) / kGruChunk), (unsigned)p.bt.batch), block(256);
  if (grid.y > 1) {
    int rc = launch_overlapped(mingru_chunk_kernel<T, true>, grid, block, 0, st, (const T*)proj, (T*)nullptr, p);
    if (rc == NQB200_OK) rc = launch_overlapped(mingru_scan_kernel, dim3((unsigned)((p.width / 2 + 63) / 64), (unsigned)p.bt.batch), dim3(64), 0, st, p);
    if (rc != NQB200_OK) return rc;
  }
  return launch_overlapped(mingru_chunk_kernel<T, false>, grid, block, 0, st, (const T*)proj, (T*)out, p);
}

template <typename T, int DPT>
static int retention_simple(const void* proj, int64_t stride, int64_t q_off, int64_t k_off, int64_t v_off, const float* decay,
                            const float* log_decay, float* state, float* o, int64_t heads, int64_t dim, int64_t vdim, const nqb200_batch* b, cudaStream_t st) {
  const dim3 grid((unsigned)((vdim + kRetCols - 1) / kRetCols), (unsigned)heads, (unsigned)b->batch), block(kRetCols * kRetGroups);
  const size_t smem = (size_t)kRetTokens * ((log_decay ? 3 : 2) * dim + kRetCols + kRetGroups * kRetCols) * sizeof(float);
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(retention_simple_kernel<T, DPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return NQB200_ERR_LAUNCH;
  }
  return launch_overlapped(retention_simple_kernel<T, DPT>, grid, block, smem, st, (const T*)proj, stride, (int)q_off, (int)k_off, (int)v_off,
                           decay, log_decay, state, o, (int)heads, (int)dim, (int)vdim, *b);
}

extern "C" int nqb200_retention(const void* proj, int64_t stride, int64_t q_off, int64_t k_off, int64_t v_off, const float* decay,
                                const float* log_decay, float* state, float* o, int64_t heads, int64_t dim, int64_t vdim, const nqb200_batch* b, int dtype,
                                void* stream) {
  const int s = check_batch(b, false);
  if (s != NQB200_OK) return s;
  if (heads <= 0 || heads > 65535 || dim <= 0 || dim > 1024 || vdim <= 0 || stride <= 0) return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (b->tokens == 0) return NQB200_OK;
  if (!proj || (!decay && !log_decay) || !state || !o) return NQB200_ERR_NULL_POINTER;
  cudaStream_t st = (cudaStream_t)stream;
#define NQB200_RET(T, D) return retention_simple<T, D>(proj, stride, q_off, k_off, v_off, decay, log_decay, state, o, heads, dim, vdim, b, st)
#define NQB200_RET_T(T)                                                                                       \
  do {                                                                                                        \
    if (dim <= 64) NQB200_RET(T, 8);                                                                          \
    if (dim <= 128) NQB200_RET(T, 16);                                                                        \
    if (dim <= 256) NQB200_RET(T, 32);                                                                        \
    if (dim <= 512) NQB200_RET(T, 64);                                                                        \
    NQB200_RET(T, 128);                                                                                       \
  } while (0)
  if (dtype == NQB200_F32) NQB200_RET_T(float);
  NQB200_RET_T(bf16);
#undef NQB200_RET_T
#undef NQB200_RET
}

extern "C" int nqb200_gla_log_decay(const void* low, int64_t low_stride, const void* a2, const float* bias, float* log_decay, int64_t tokens,
                                    int64_t channels, int64_t rank, float tau, int dtype, void* stream) {
  if (tokens < 0 || channels <= 0 || channels > INT32_MAX || rank <= 0 || rank > 512 || low_stride < rank || !(tau > 0.f)) return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (tokens == 0) return NQB200_OK;
  if (!low || !a2 || !bias || !log_decay) return NQB200_ERR_NULL_POINTER;
  const int64_t ty = (tokens + kDecayTokens - 1) / kDecayTokens;
  if (ty > 65535) return NQB200_ERR_TOO_LARGE;
  const dim3 grid((unsigned)((channels + 255) / 256), (unsigned)ty), block(256);
  const size_t smem = (size_t)kDecayTokens * rank * sizeof(float);
  if (dtype == NQB200_F32)
    return launch_overlapped(gla_log_decay_kernel<float>, grid, block, smem, (cudaStream_t)stream, (const float*)low, low_stride, (const float*)a2, bias,
                             log_decay, tokens, (int)channels, (int)rank, 1.f / tau);
  return launch_overlapped(gla_log_decay_kernel<bf16>, grid, block, smem, (cudaStream_t)stream, (const bf16*)low, low_stride, (const bf16*)a2, bias,
                           log_decay, tokens, (int)channels, (int)rank, 1.f / tau);
}

extern "C" int nqb200_head_norm_gate(const float* o, const void* gate, int64_t gate_stride, const float* weight, void* out, int64_t out_stride, int64_t tokens,
                                     int64_t heads, int64_t vdim, float eps, float out_scale, int dtype, void* stream) {
  if (tokens < 0 || heads <= 0 || vdim <= 0) return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (tokens == 0) return NQB200_OK;
  if (!o || !gate || !out) return NQB200_ERR_NULL_POINTER;
  const int64_t pairs = tokens * heads;
  const dim3 grid((unsigned)((pairs + 7) / 8)), block(256);
  if (dtype == NQB200_F32)
    return launch_overlapped(head_norm_gate_kernel<float>, grid, block, 0, (cudaStream_t)stream, o, (const float*)gate, gate_stride, weight, (float*)out,
                             out_stride, pairs, (int)heads, (int)vdim, eps, out_scale);
  return launch_overlapped(head_norm_gate_kernel<bf16>, grid, block, 0, (cudaStream_t)stream, o, (const bf16*)gate, gate_stride, weight, (bf16*)out,
                           out_stride, pairs, (int)heads, (int)vdim, eps, out_scale);
}

extern "C" int64_t nqb200_mingru_scratch(int64_t tokens, int64_t batch, int64_t width) {
  return (tokens / kGruChunk + batch) * width * 2;
}

extern "C" int nqb200_mingru(const void* proj, int64_t stride, int64_t z_off, int64_t x_off, int64_t g_off, const float* z_bias,
                             const float* x_bias, float* state, void* out, int64_t width, float* scratch, const nqb200_batch* b, int dtype,
                             void* stream) {
  const int s = check_batch(b, false);
  if (s != NQB200_OK) return s;
  if (width <= 0 || width > INT32_MAX || stride <= 0) return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (b->tokens == 0) return NQB200_OK;
  if (!proj || !z_bias || !x_bias || !state || !out) return NQB200_ERR_NULL_POINTER;
  cudaStream_t st = (cudaStream_t)stream;
  const bool pairs = width % 2 == 0 && stride % 2 == 0 && z_off % 2 == 0 && x_off % 2 == 0 && g_off % 2 == 0 && aligned16(proj) && aligned16(out) &&
                     aligned16(z_bias) && aligned16(x_bias) && aligned16(state);
  if (pairs && b->max_len > 1 && (b->max_len + kGruChunk - 1) / kGruChunk <= 65535) {
    if (b->max_len > kGruChunk && (!scratch || !aligned16(scratch))) return NQB200_ERR_WORKSPACE;
    GruArgs p = {};
    p.stride = stride; p.z_off = (int)z_off; p.x_off = (int)x_off; p.g_off = (int)g_off; p.width = (int)width;
    p.z_bias = z_bias; p.x_bias = x_bias; p.state = state; p.bt = *b;
    p.folds = reinterpret_cast<float2*>(scratch);
    return dtype == NQB200_F32 ? mingru_chunked<float>(proj, out, p, st) : mingru_chunked<bf16>(proj, out, p, st);
  }
  const dim3 grid((unsigned)((width + kGruCols - 1) / kGruCols), (unsigned)b->batch), block(kGruSegs * kGruCols);
  if (dtype == NQB200_F32)
    return launch_overlapped(mingru_kernel<float>, grid, block, 0, st, (const float*)proj, stride, (int)z_off, (int)x_off, (int)g_off, z_bias,
                             x_bias, state, (float*)out, (int)width, *b);
  return launch_overlapped(mingru_kernel<bf16>, grid, block, 0, st, (const bf16*)proj, stride, (int)z_off, (int)x_off, (int)g_off, z_bias, x_bias,
                           state, (bf16*)out, (int)width, *b);
}
