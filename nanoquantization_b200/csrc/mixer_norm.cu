// The residual stream's own steps: embedding / loop entry, RMS norm, RMS norm + input convolution, norms after the
// residual sum, per-layer token inputs, and the clamped GLU between the feed-forward's linears.  The stream is float; a
// norm reads it once and leaves the 16-bit operand of the next linear.
#include "mixers.cuh"

namespace nqb200 {

template <typename T>
__global__ void __launch_bounds__(256) stream_add_kernel(float* __restrict__ x, const int64_t* __restrict__ ids,
                                                         const T* __restrict__ embed, const float* __restrict__ step,
                                                         int accumulate, int width) {
  grid_launch_dependents();
  grid_dependency_wait();
  float* row = x + (size_t)blockIdx.x * width;
  const T* e = ids ? embed + (size_t)ids[blockIdx.x] * width : nullptr;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    float v = accumulate ? row[c] : 0.f;
    if (e) v += to_f(e[c]);
    if (step) v += step[c];
    row[c] = v;
  }
}

template <typename T>
__global__ void __launch_bounds__(256) rmsnorm_rows_kernel(const float* __restrict__ x, const int64_t* __restrict__ rows,
                                                           const float* __restrict__ weight, T* __restrict__ out, int width, float eps) {
  __shared__ float red[8];
  grid_launch_dependents();
  grid_dependency_wait();
  const float* row = x + (size_t)(rows ? rows[blockIdx.x] : blockIdx.x) * width;
  float ss = 0.f;
  for (int c = threadIdx.x; c < width; c += 256) ss += row[c] * row[c];
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) tot += red[w];
  const float inv = 1.f / sqrtf(tot / (float)width + eps);
  for (int c = threadIdx.x; c < width; c += 256) out[(size_t)blockIdx.x * width + c] = from_f<T>(row[c] * inv * weight[c]);
}

// A CTA takes `tile` tokens of one sequence (tile >= taps - 1).  It needs 1/rms of those and of the taps - 1
// tokens before them; rows from before this step come from the state, which only the first tile of a sequence
// reaches.  That same CTA also writes the new state (it recomputes the norm of the step's last taps - 1 tokens),
// so the state is read and written by one CTA and no order between CTAs matters.
template <typename T>
__global__ void __launch_bounds__(256) rmsnorm_conv_kernel(const float* __restrict__ x, const float* __restrict__ weight,
                                                           const float* __restrict__ conv, float* state, T* __restrict__ out,
                                                           const nqb200_batch bt, int width, int taps, int tile, float eps) {
  extern __shared__ float inv_s[];  // [halo + tile] tokens around the tile, then [halo] last tokens of the step
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.y, t0 = bt.cu[b], n = bt.cu[b + 1] - t0, first = blockIdx.x * tile;
  if (first >= n) return;
  const int halo = taps - 1, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
  const bool head = first == 0;
  for (int r = warp; r < halo + tile + (head ? halo : 0); r += nwarps) {
    const int tok = r < halo + tile ? first - halo + r : n - halo + (r - halo - tile);
    if (tok < 0 || tok >= n) continue;
    const float* row = x + (size_t)(t0 + tok) * width;
    float ss = 0.f;
    for (int c = lane; c < width; c += 32) ss += row[c] * row[c];
    ss = warp_sum(ss);
    if (lane == 0) inv_s[r] = 1.f / sqrtf(ss / (float)width + eps);
  }
  __syncthreads();
  const bool fresh = bt.pos0[b] == 0;
  float* st = state + (size_t)bt.slot[b] * halo * width;
  const int cnt = min(tile, n - first);
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float w = weight[c];
    for (int i = 0; i < cnt; ++i) {
      const int tok = first + i;
      const float h = x[(size_t)(t0 + tok) * width + c] * inv_s[halo + i] * w;
      float acc = 0.f;
      for (int j = 0; j < halo; ++j) {
        const int src = tok - halo + j;
        float hv = 0.f;
        if (src >= 0) hv = x[(size_t)(t0 + src) * width + c] * inv_s[i + j] * w;
        else if (!fresh) hv = st[(size_t)(src + halo) * width + c];
        acc += conv[(size_t)j * width + c] * hv;
      }
      acc += conv[(size_t)halo * width + c] * h;
      out[(size_t)(t0 + tok) * width + c] = from_f<T>(h + acc);
    }
    if (head) {
      for (int r = 0; r < halo; ++r) {  // ascending: an old row that moves down is read before it is overwritten
        const int src = n - halo + r;
        float hv = 0.f;
        if (src >= 0) hv = x[(size_t)(t0 + src) * width + c] * inv_s[halo + tile + r] * w;
        else if (!fresh) hv = st[(size_t)(src + halo) * width + c];
        st[(size_t)r * width + c] = hv;
      }
    }
  }
}

template <typename T> __device__ __forceinline__ void store4(T* p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store4<bf16>(bf16* p, float4 v) {
  uint2 r;
  r.x = (uint32_t)__bfloat16_as_ushort(__float2bfloat16_rn(v.x)) | ((uint32_t)__bfloat16_as_ushort(__float2bfloat16_rn(v.y)) << 16);
  r.y = (uint32_t)__bfloat16_as_ushort(__float2bfloat16_rn(v.z)) | ((uint32_t)__bfloat16_as_ushort(__float2bfloat16_rn(v.w)) << 16);
  *reinterpret_cast<uint2*>(p) = r;
}
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const float* p) { return ld4(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(r.x << 16), __uint_as_float(r.x & 0xFFFF0000u), __uint_as_float(r.y << 16), __uint_as_float(r.y & 0xFFFF0000u));
}
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float4 scale4(float4 a, float s) { return make_float4(a.x * s, a.y * s, a.z * s, a.w * s); }
__device__ __forceinline__ void fma4(float4& d, float4 a, float4 b) { d.x += a.x * b.x; d.y += a.y * b.y; d.z += a.z * b.z; d.w += a.w * b.w; }

// The same for widths that are multiples of 4 and short filters: float4 accesses, and the last taps - 1 rows of h
// stay in registers while a thread walks down the tile's tokens.
constexpr int kConvTile = 16;
template <typename T, int TAPS>
__global__ void __launch_bounds__(256) rmsnorm_conv_vec_kernel(const float* __restrict__ x, const float* __restrict__ weight,
                                                               const float* __restrict__ conv, float* state, T* __restrict__ out,
                                                               const nqb200_batch bt, int width, float eps) {
  constexpr int HALO = TAPS - 1;
  __shared__ float inv_s[kConvTile + 2 * HALO];
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.y, t0 = bt.cu[b], n = bt.cu[b + 1] - t0, first = blockIdx.x * kConvTile;
  if (first >= n) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool head = first == 0;
  for (int r = warp; r < kConvTile + HALO + (head ? HALO : 0); r += 8) {
    const int tok = r < kConvTile + HALO ? first - HALO + r : n - HALO + (r - HALO - kConvTile);
    if (tok < 0 || tok >= n) continue;
    const float* row = x + (size_t)(t0 + tok) * width;
    float ss = 0.f;
    for (int c = lane * 4; c < width; c += 128) {
      const float4 v = ld4(row + c);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    ss = warp_sum(ss);
    if (lane == 0) inv_s[r] = 1.f / sqrtf(ss / (float)width + eps);
  }
  __syncthreads();
  const bool fresh = bt.pos0[b] == 0;
  float* st = state + (size_t)bt.slot[b] * HALO * width;
  const int cnt = min(kConvTile, n - first);
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int c = threadIdx.x * 4; c < width; c += 1024) {
    const float4 w = ld4(weight + c);
    float4 cw[TAPS], win[HALO];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) cw[j] = ld4(conv + (size_t)j * width + c);
    float4 old[HALO];   // the state as it was: read whole before it is written
#pragma unroll
    for (int j = 0; j < HALO; ++j) old[j] = (head && !fresh) ? ld4(st + (size_t)j * width + c) : zero;
#pragma unroll
    for (int j = 0; j < HALO; ++j) {
      const int src = first - HALO + j;
      win[j] = src >= 0 ? mul4(scale4(ld4(x + (size_t)(t0 + src) * width + c), inv_s[j]), w) : old[j];
    }
#pragma unroll 4
    for (int i = 0; i < cnt; ++i) {
      const float4 h = mul4(scale4(ld4(x + (size_t)(t0 + first + i) * width + c), inv_s[HALO + i]), w);
      float4 acc = h;
#pragma unroll
      for (int j = 0; j < HALO; ++j) fma4(acc, cw[j], win[j]);
      fma4(acc, cw[HALO], h);
      store4<T>(out + (size_t)(t0 + first + i) * width + c, acc);
#pragma unroll
      for (int j = 0; j + 1 < HALO; ++j) win[j] = win[j + 1];
      win[HALO - 1] = h;
    }
    if (head) {
#pragma unroll
      for (int r = 0; r < HALO; ++r) {
        const int src = n - HALO + r;
        float4 hv = zero;
        if (src >= 0) {
          hv = mul4(scale4(ld4(x + (size_t)(t0 + src) * width + c), inv_s[HALO + kConvTile + r]), w);
        } else {
#pragma unroll
          for (int j = 0; j < HALO; ++j)
            if (j == src + HALO) hv = old[j];
        }
        *reinterpret_cast<float4*>(st + (size_t)r * width + c) = hv;
      }
    }
  }
}

// One token per sequence: a CTA takes the token, the row stays in shared memory between the sum of squares and the use.
template <typename T>
__global__ void __launch_bounds__(512) rmsnorm_conv_decode_kernel(const float* __restrict__ x, const float* __restrict__ weight,
                                                                  const float* __restrict__ conv, float* state, T* __restrict__ out,
                                                                  const nqb200_batch bt, int width, int taps, float eps) {
  extern __shared__ float4 row_s[];
  __shared__ float red[16];
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.x, t0 = bt.cu[b];
  if (bt.cu[b + 1] == t0) return;
  const int halo = taps - 1;
  const float* row = x + (size_t)t0 * width;
  float* st = state + (size_t)bt.slot[b] * halo * width;
  const bool fresh = bt.pos0[b] == 0;
  float ss = 0.f;
  for (int c = threadIdx.x; c * 4 < width; c += 512) {
    const float4 v = ld4(row + c * 4);
    row_s[c] = v;
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < 16; ++w) tot += red[w];
  const float inv = 1.f / sqrtf(tot / (float)width + eps);
  for (int c = threadIdx.x * 4; c < width; c += 2048) {
    const float4 h = mul4(scale4(row_s[c / 4], inv), ld4(weight + c));
    float4 acc = h;
    fma4(acc, ld4(conv + (size_t)halo * width + c), h);
    for (int j = 0; j < halo; ++j) {
      const float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : ld4(st + (size_t)j * width + c);
      fma4(acc, ld4(conv + (size_t)j * width + c), s);
      if (j > 0) *reinterpret_cast<float4*>(st + (size_t)(j - 1) * width + c) = s;
    }
    if (halo > 0) *reinterpret_cast<float4*>(st + (size_t)(halo - 1) * width + c) = h;
    store4<T>(out + (size_t)t0 * width + c, acc);
  }
}

template <typename T>
static int launch_rmsnorm_conv(const float* x, const float* weight, const float* conv, float* state, T* out, const nqb200_batch* b,
                               int width, int taps, float eps, cudaStream_t st) {
  const bool vec = width % 4 == 0 && aligned16(x) && aligned16(weight) && aligned16(conv) && aligned16(out) && (!state || aligned16(state));
  if (vec && b->max_len == 1 && width <= 8192) {
    return launch_overlapped(rmsnorm_conv_decode_kernel<T>, dim3((unsigned)b->batch), dim3(512), (size_t)width * 4, st, x, weight, conv, state, out,
                             *b, width, taps, eps);
  }
  const dim3 block(256);
  if (vec && taps >= 2 && taps <= 5) {
    const dim3 grid((unsigned)((b->max_len + kConvTile - 1) / kConvTile), (unsigned)b->batch);
#define NQB200_CONV(K) return launch_overlapped(rmsnorm_conv_vec_kernel<T, K>, grid, block, 0, st, x, weight, conv, state, out, *b, width, eps)
    if (taps == 2) NQB200_CONV(2);
    if (taps == 3) NQB200_CONV(3);
    if (taps == 4) NQB200_CONV(4);
    NQB200_CONV(5);
#undef NQB200_CONV
  }
  const int halo = taps - 1, tile = halo > 8 ? halo : 8;
  const dim3 grid((unsigned)((b->max_len + tile - 1) / tile), (unsigned)b->batch);
  return launch_overlapped(rmsnorm_conv_kernel<T>, grid, block, (size_t)(2 * halo + tile) * sizeof(float), st, x, weight, conv, state, out, *b,
                           width, taps, tile, eps);
}

// Norms after the sum.  A CTA takes a token; the row (alpha x + the terms of y) stays in shared memory between the sums of
// squares and the use.  The groups of the row are split into about as many pieces as there are warps, a warp sums whole
// pieces, and the group's scale is taken from its pieces.  out: the row rounded to T; x (if written): the row itself.
// Few rows: wide CTAs, so that a row's loads (of every term) are under way at once.
constexpr int kNormThreads = 256, kNormWarps = kNormThreads / 32, kNormWide = 1024;
template <typename T, typename Y, int THREADS>
__global__ void __launch_bounds__(THREADS, THREADS == kNormWide ? 1 : 4) group_norm_kernel(float* x, const int64_t* __restrict__ rows, const Y* __restrict__ y, int terms, float alpha,
                                                                  const float* __restrict__ weight, T* __restrict__ out, int width, int groups, int pieces,
                                                                  float eps, int write_x) {
  extern __shared__ float4 norm_smem[];
  float* row_s = reinterpret_cast<float*>(norm_smem);        // [width]
  float* part = row_s + (width + 3) / 4 * 4;                 // [groups * pieces]
  grid_launch_dependents();
  grid_dependency_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  constexpr int threads = THREADS, U = THREADS == kNormWide ? 8 : 4;   // terms under way at once
  const int64_t at = rows ? rows[blockIdx.x] : blockIdx.x;
  float* xr = x + (size_t)at * width;
  const Y* yr = y + (size_t)blockIdx.x * terms * width;
  const int size = width / groups;
  const bool vec = size % 4 == 0;
  if (vec) {
    for (int c = tid * 4; c < width; c += threads * 4) {
      float4 v = scale4(ld4(xr + c), alpha);
      for (int j0 = 0; j0 < terms; j0 += U) {
        float4 a[U];
#pragma unroll
        for (int j = 0; j < U; ++j) a[j] = j0 + j < terms ? load4(yr + (size_t)(j0 + j) * width + c) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int j = 0; j < U; ++j) { v.x += a[j].x; v.y += a[j].y; v.z += a[j].z; v.w += a[j].w; }
      }
      *reinterpret_cast<float4*>(row_s + c) = v;
    }
  } else {
    for (int c = tid; c < width; c += threads) {
      float v = alpha * xr[c];
      for (int j = 0; j < terms; ++j) v += to_f(yr[(size_t)j * width + c]);
      row_s[c] = v;
    }
  }
  __syncthreads();
  const int len = (size + pieces - 1) / pieces;
  for (int q = warp; q < groups * pieces; q += threads / 32) {
    const int g = q / pieces, lo = (q - g * pieces) * len, hi = min(lo + len, size);
    const float* s = row_s + g * size;
    float ss = 0.f;
    for (int c = lo + lane; c < hi; c += 32) ss += s[c] * s[c];
    ss = warp_sum(ss);
    if (lane == 0) part[q] = ss;
  }
  __syncthreads();
  for (int g = tid; g < groups; g += threads) {   // a thread per group; its pieces' places become free for the scale
    float ss = 0.f;
    for (int k = 0; k < pieces; ++k) ss += part[g * pieces + k];
    part[g * pieces] = 1.f / sqrtf(ss / (float)size + eps);
  }
  __syncthreads();
  T* o = out + (size_t)blockIdx.x * width;
  if (vec) {
    for (int c = tid * 4; c < width; c += threads * 4) {
      const float4 v = mul4(scale4(*reinterpret_cast<const float4*>(row_s + c), part[c / size * pieces]), ld4(weight + c));
      if (write_x) *reinterpret_cast<float4*>(xr + c) = v;
      store4<T>(o + c, v);
    }
  } else {
    for (int c = tid; c < width; c += threads) {
      const float v = row_s[c] * part[c / size * pieces] * weight[c];
      if (write_x) xr[c] = v;
      o[c] = from_f<T>(v);
    }
  }
}

// x += y / rms(y) * weight, and the sum rounded to T.
template <typename T>
__global__ void __launch_bounds__(kNormThreads) add_normed_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ weight,
                                                                  T* __restrict__ out, int width, float eps) {
  __shared__ float red[kNormWarps];
  grid_launch_dependents();
  grid_dependency_wait();
  float* xr = x + (size_t)blockIdx.x * width;
  const float* yr = y + (size_t)blockIdx.x * width;
  T* o = out + (size_t)blockIdx.x * width;
  const int tid = threadIdx.x;
  const bool vec = width % 4 == 0;
  float ss = 0.f;
  if (vec) {
    for (int c = tid * 4; c < width; c += kNormThreads * 4) { const float4 v = ld4(yr + c); ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
  } else {
    for (int c = tid; c < width; c += kNormThreads) ss += yr[c] * yr[c];
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < kNormWarps; ++w) tot += red[w];
  const float inv = 1.f / sqrtf(tot / (float)width + eps);
  if (vec) {
    for (int c = tid * 4; c < width; c += kNormThreads * 4) {
      float4 v = ld4(xr + c);
      fma4(v, scale4(ld4(yr + c), inv), ld4(weight + c));
      *reinterpret_cast<float4*>(xr + c) = v;
      store4<T>(o + c, v);
    }
  } else {
    for (int c = tid; c < width; c += kNormThreads) {
      const float v = xr[c] + yr[c] * inv * weight[c];
      xr[c] = v;
      o[c] = from_f<T>(v);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) gelu_table_kernel(const T* __restrict__ gate, const int64_t* __restrict__ ids, const T* __restrict__ table,
                                                         int64_t table_stride, T* __restrict__ out, int64_t tokens, int dim) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int64_t total = tokens * (int64_t)dim;
  for (int64_t e = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; e < total; e += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = e / dim, i = e - t * dim;
    out[e] = from_f<T>(gelu_tanh_f(to_f(gate[e])) * to_f(table[ids[t] * table_stride + i]));
  }
}

template <typename T, typename Y, int THREADS>
static int launch_group_norm_by(float* x, const int64_t* rows, const void* y, int64_t terms, float alpha, const float* weight, void* out, int64_t n,
                             int64_t width, int64_t groups, float eps, int write_x, cudaStream_t st) {
  constexpr int warps = THREADS / 32;
  const int pieces = groups >= warps ? 1 : (int)((warps + groups - 1) / groups);
  const size_t smem = ((size_t)(width + 3) / 4 * 4 + (size_t)groups * pieces) * sizeof(float);
  if (smem > 200 * 1024) return NQB200_ERR_TOO_LARGE;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(group_norm_kernel<T, Y, THREADS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return NQB200_ERR_LAUNCH;
  }
  return launch_overlapped(group_norm_kernel<T, Y, THREADS>, dim3((unsigned)n), dim3(THREADS), smem, st, x, rows, (const Y*)y, (int)terms, alpha, weight,
                           (T*)out, (int)width, (int)groups, pieces, eps, write_x);
}

template <typename T, typename Y>
static int launch_group_norm(float* x, const int64_t* rows, const void* y, int64_t terms, float alpha, const float* weight, void* out, int64_t n,
                             int64_t width, int64_t groups, float eps, int write_x, cudaStream_t st) {
  if (n <= 2 * kNumSMs && width > 2 * kNormThreads)
    return launch_group_norm_by<T, Y, kNormWide>(x, rows, y, terms, alpha, weight, out, n, width, groups, eps, write_x, st);
  return launch_group_norm_by<T, Y, kNormThreads>(x, rows, y, terms, alpha, weight, out, n, width, groups, eps, write_x, st);
}

template <typename T>
__global__ void __launch_bounds__(256) clamped_glu_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int64_t tokens, int ff,
                                                          float limit) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int64_t total = tokens * (int64_t)ff;
  for (int64_t idx = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; idx < total; idx += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = idx / ff, i = idx - t * ff;
    const float g = fminf(to_f(gate_up[t * 2 * ff + i]), limit);
    const float u = fminf(fmaxf(to_f(gate_up[t * 2 * ff + ff + i]), -limit), limit);
    out[idx] = from_f<T>(g * sigmoid_f(1.702f * g) * (u + 1.f));
  }
}

// The same, 8 values per thread and bf16.
__global__ void __launch_bounds__(256) clamped_glu_vec_kernel(const bf16* __restrict__ gate_up, bf16* __restrict__ out, int64_t tokens, int ff8, float limit) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int64_t total = tokens * (int64_t)ff8;
  for (int64_t idx = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; idx < total; idx += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = idx / ff8, i = idx - t * ff8;
    const uint4 gv = reinterpret_cast<const uint4*>(gate_up)[t * 2 * ff8 + i], uv = reinterpret_cast<const uint4*>(gate_up)[t * 2 * ff8 + ff8 + i];
    const uint32_t gw[4] = {gv.x, gv.y, gv.z, gv.w}, uw[4] = {uv.x, uv.y, uv.z, uv.w};
    uint32_t ow[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      float y[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float g = fminf(__uint_as_float(e ? gw[k] & 0xFFFF0000u : gw[k] << 16), limit);
        const float u = fminf(fmaxf(__uint_as_float(e ? uw[k] & 0xFFFF0000u : uw[k] << 16), -limit), limit);
        y[e] = g * sigmoid_fast(1.702f * g) * (u + 1.f);
      }
      ow[k] = (uint32_t)__bfloat16_as_ushort(__float2bfloat16_rn(y[0])) | ((uint32_t)__bfloat16_as_ushort(__float2bfloat16_rn(y[1])) << 16);
    }
    reinterpret_cast<uint4*>(out)[idx] = make_uint4(ow[0], ow[1], ow[2], ow[3]);
  }
}

}  // namespace nqb200

using namespace nqb200;

extern "C" int nqb200_stream_add(float* x, const int64_t* ids, const void* embed, const float* step, int accumulate, int64_t tokens,
                                 int64_t width, int dtype, void* stream) {
  if (tokens < 0 || width <= 0 || tokens > INT32_MAX || width > INT32_MAX) return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (tokens == 0) return NQB200_OK;
  if (!x || (ids && !embed)) return NQB200_ERR_NULL_POINTER;
  const dim3 grid((unsigned)tokens), block(256);
  if (dtype == NQB200_F32)
    return launch_overlapped(stream_add_kernel<float>, grid, block, 0, (cudaStream_t)stream, x, ids, (const float*)embed, step, accumulate, (int)width);
  return launch_overlapped(stream_add_kernel<bf16>, grid, block, 0, (cudaStream_t)stream, x, ids, (const bf16*)embed, step, accumulate, (int)width);
}

extern "C" int nqb200_rmsnorm_rows(const float* x, const int64_t* rows, const float* weight, void* out, int64_t n_rows, int64_t width,
                                   float eps, int dtype, void* stream) {
  if (n_rows < 0 || width <= 0 || n_rows > INT32_MAX || width > INT32_MAX) return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (n_rows == 0) return NQB200_OK;
  if (!x || !weight || !out) return NQB200_ERR_NULL_POINTER;
  const dim3 grid((unsigned)n_rows), block(256);
  if (dtype == NQB200_F32)
    return launch_overlapped(rmsnorm_rows_kernel<float>, grid, block, 0, (cudaStream_t)stream, x, rows, weight, (float*)out, (int)width, eps);
  return launch_overlapped(rmsnorm_rows_kernel<bf16>, grid, block, 0, (cudaStream_t)stream, x, rows, weight, (bf16*)out, (int)width, eps);
}

static int group_norm_shape(int64_t n, int64_t width, int64_t groups, int dtype) {
  if (n < 0 || width <= 0 || n > INT32_MAX || width > INT32_MAX || groups <= 0 || width % groups != 0) return NQB200_ERR_BAD_SHAPE;
  return mixer_dtype(dtype) ? NQB200_OK : NQB200_ERR_BAD_DTYPE;
}

extern "C" int nqb200_group_norm_rows(const float* x, const int64_t* rows, const float* weight, void* out, int64_t n_rows, int64_t width, int64_t groups,
                                      float eps, int dtype, void* stream) {
  const int s = group_norm_shape(n_rows, width, groups, dtype);
  if (s != NQB200_OK || n_rows == 0) return s;
  if (!x || !weight || !out) return NQB200_ERR_NULL_POINTER;
  if (!aligned16(x) || !aligned16(weight) || !aligned16(out)) return NQB200_ERR_MISALIGNED;
  cudaStream_t st = (cudaStream_t)stream;
  float* xs = const_cast<float*>(x);   // not written
  if (dtype == NQB200_F32) return launch_group_norm<float, float>(xs, rows, nullptr, 0, 1.f, weight, out, n_rows, width, groups, eps, 0, st);
  return launch_group_norm<bf16, float>(xs, rows, nullptr, 0, 1.f, weight, out, n_rows, width, groups, eps, 0, st);
}

extern "C" int nqb200_post_norm(float* x, const void* y, int y_dtype, int64_t terms, float alpha, const float* weight, void* h, int64_t tokens,
                                int64_t width, int64_t groups, float eps, int dtype, void* stream) {
  const int s = group_norm_shape(tokens, width, groups, dtype);
  if (s != NQB200_OK) return s;
  if (terms < 0 || terms > INT32_MAX) return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(y_dtype)) return NQB200_ERR_BAD_DTYPE;
  if (tokens == 0) return NQB200_OK;
  if (!x || !weight || !h || (terms > 0 && !y)) return NQB200_ERR_NULL_POINTER;
  if (!aligned16(x) || !aligned16(weight) || !aligned16(h) || !aligned16(y)) return NQB200_ERR_MISALIGNED;
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == NQB200_F32)
    return y_dtype == NQB200_F32 ? launch_group_norm<float, float>(x, nullptr, y, terms, alpha, weight, h, tokens, width, groups, eps, 1, st)
                                 : launch_group_norm<float, bf16>(x, nullptr, y, terms, alpha, weight, h, tokens, width, groups, eps, 1, st);
  return y_dtype == NQB200_F32 ? launch_group_norm<bf16, float>(x, nullptr, y, terms, alpha, weight, h, tokens, width, groups, eps, 1, st)
                               : launch_group_norm<bf16, bf16>(x, nullptr, y, terms, alpha, weight, h, tokens, width, groups, eps, 1, st);
}

extern "C" int nqb200_gelu_table(const void* gate, const int64_t* ids, const void* table, int64_t table_stride, int64_t column, void* out, int64_t tokens,
                                 int64_t dim, int dtype, void* stream) {
  if (tokens < 0 || dim <= 0 || dim > INT32_MAX || column < 0 || table_stride < column + dim) return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (tokens == 0) return NQB200_OK;
  if (!gate || !ids || !table || !out) return NQB200_ERR_NULL_POINTER;
  const int64_t want = (tokens * dim + 255) / 256;
  const dim3 grid((unsigned)(want < (int64_t)kNumSMs * 16 ? want : (int64_t)kNumSMs * 16)), block(256);
  if (dtype == NQB200_F32)
    return launch_overlapped(gelu_table_kernel<float>, grid, block, 0, (cudaStream_t)stream, (const float*)gate, ids, (const float*)table + column,
                             table_stride, (float*)out, tokens, (int)dim);
  return launch_overlapped(gelu_table_kernel<bf16>, grid, block, 0, (cudaStream_t)stream, (const bf16*)gate, ids, (const bf16*)table + column, table_stride,
                           (bf16*)out, tokens, (int)dim);
}

extern "C" int nqb200_add_normed(float* x, const float* y, const float* weight, void* h, int64_t tokens, int64_t width, float eps, int dtype,
                                 void* stream) {
  const int s = group_norm_shape(tokens, width, 1, dtype);
  if (s != NQB200_OK || tokens == 0) return s;
  if (!x || !y || !weight || !h) return NQB200_ERR_NULL_POINTER;
  if (!aligned16(x) || !aligned16(y) || !aligned16(weight) || !aligned16(h)) return NQB200_ERR_MISALIGNED;
  const dim3 grid((unsigned)tokens), block(kNormThreads);
  if (dtype == NQB200_F32)
    return launch_overlapped(add_normed_kernel<float>, grid, block, 0, (cudaStream_t)stream, x, y, weight, (float*)h, (int)width, eps);
  return launch_overlapped(add_normed_kernel<bf16>, grid, block, 0, (cudaStream_t)stream, x, y, weight, (bf16*)h, (int)width, eps);
}

extern "C" int nqb200_rmsnorm_conv(const float* x, const float* weight, const float* conv, float* state, void* out,
                                   const nqb200_batch* b, int64_t width, int64_t taps, float eps, int dtype, void* stream) {
  const int st = check_batch(b, false);
  if (st != NQB200_OK) return st;
  if (width <= 0 || width > INT32_MAX || taps <= 0 || taps > 1024) return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (b->tokens == 0) return NQB200_OK;
  if (!x || !weight || !conv || !out || (taps > 1 && !state)) return NQB200_ERR_NULL_POINTER;
  if (dtype == NQB200_F32)
    return launch_rmsnorm_conv<float>(x, weight, conv, state, (float*)out, b, (int)width, (int)taps, eps, (cudaStream_t)stream);
  return launch_rmsnorm_conv<bf16>(x, weight, conv, state, (bf16*)out, b, (int)width, (int)taps, eps, (cudaStream_t)stream);
}

extern "C" int nqb200_clamped_glu(const void* gate_up, void* out, int64_t tokens, int64_t ff, float limit, int dtype, void* stream) {
  if (tokens < 0 || ff <= 0 || ff > INT32_MAX) return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (tokens == 0) return NQB200_OK;
  if (!gate_up || !out) return NQB200_ERR_NULL_POINTER;
  if (dtype == NQB200_BF16 && ff % 8 == 0 && aligned16(gate_up) && aligned16(out)) {
    const int64_t blocks = (tokens * (ff / 8) + 255) / 256;
    return launch_overlapped(clamped_glu_vec_kernel, dim3((unsigned)(blocks < INT32_MAX ? blocks : INT32_MAX)), dim3(256), 0, (cudaStream_t)stream,
                             (const bf16*)gate_up, (bf16*)out, tokens, (int)(ff / 8), limit);
  }
  const int64_t want = (tokens * ff + 255) / 256;
  const dim3 grid((unsigned)(want < (int64_t)kNumSMs * 16 ? want : (int64_t)kNumSMs * 16)), block(256);
  if (dtype == NQB200_F32)
    return launch_overlapped(clamped_glu_kernel<float>, grid, block, 0, (cudaStream_t)stream, (const float*)gate_up, (float*)out, tokens, (int)ff, limit);
  return launch_overlapped(clamped_glu_kernel<bf16>, grid, block, 0, (cudaStream_t)stream, (const bf16*)gate_up, (bf16*)out, tokens, (int)ff, limit);
}
