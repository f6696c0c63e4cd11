// Rotary embedding + paged K/V store, and attention (chunks, score cap and sink, or sigmoid weights).  The kernels in
// this file take any head sizes and both element types; the tensor-core kernels take over where they apply.
#include "mixers.cuh"

namespace nqb200 {

// One CTA per token: the token's cos / sin once into shared memory, then every head of q, k and v.
template <typename T>
__global__ void __launch_bounds__(256) rope_store_kernel(T* __restrict__ proj, T* __restrict__ k_cache, T* __restrict__ v_cache,
                                                         const float* __restrict__ inv_freq, const nqb200_batch bt, int stride, int q_off,
                                                         int k_off, int v_off, int heads, int kv_heads, int dim, int vdim, int rot) {
  extern __shared__ float cs[];  // [rot/2] cos, [rot/2] sin
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.y, i = blockIdx.x, t0 = bt.cu[b];
  if (i >= bt.cu[b + 1] - t0) return;
  const int p = bt.pos0[b] + i, half = rot / 2;
  for (int f = threadIdx.x; f < half; f += blockDim.x) sincosf((float)p * inv_freq[f], &cs[half + f], &cs[f]);
  __syncthreads();
  T* row = proj + (size_t)(t0 + i) * stride;
  const size_t slot = kv_row(bt, b, p);
  T* kd = k_cache + slot * kv_heads * dim;
  T* vd = v_cache + slot * kv_heads * vdim;
  const int per = half + (dim - rot);  // rotation pairs, then the dimensions that pass
  for (int e = threadIdx.x; e < (heads + kv_heads) * per; e += blockDim.x) {
    const int hd = e / per, j = e - hd * per;
    const bool isq = hd < heads;
    const T* src = row + (isq ? q_off + hd * dim : k_off + (hd - heads) * dim);
    T* dst = isq ? row + q_off + hd * dim : kd + (hd - heads) * dim;
    if (j < half) {
      const float u = to_f(src[j]), v = to_f(src[j + half]), c = cs[j], s = cs[half + j];
      dst[j] = from_f<T>(u * c - v * s);
      dst[j + half] = from_f<T>(v * c + u * s);
    } else if (!isq) {
      dst[j + half] = src[j + half];
    }
  }
  for (int e = threadIdx.x; e < kv_heads * vdim; e += blockDim.x) vd[e] = row[v_off + e];
}

// One CTA per token and a warp per head: optional RMS norm of the head, rotation in either pair layout, store.
template <typename T>
__global__ void __launch_bounds__(256) norm_rope_kernel(T* __restrict__ proj, T* __restrict__ k_cache, T* __restrict__ v_cache, const nqb200_rope r,
                                                        const nqb200_batch bt, int64_t stride, int q_off, int k_off, int v_off) {
  extern __shared__ float cs[];  // [rot/2] cos, [rot/2] sin
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.y, i = blockIdx.x, t0 = bt.cu[b], half = r.rot / 2, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (i >= bt.cu[b + 1] - t0) return;
  const int p = bt.pos0[b] + i;
  for (int f = threadIdx.x; f < half; f += blockDim.x) sincosf((float)p * r.inv_freq[f], &cs[half + f], &cs[f]);
  __syncthreads();
  T* row = proj + (size_t)(t0 + i) * stride;
  const size_t slot = k_cache ? kv_row(bt, b, p) : 0;
  const int first = r.interleaved ? 1 : half, step = r.interleaved ? 2 : 1;   // distance inside a pair, and between pairs
  for (int hd = warp; hd < r.heads + r.kv_heads; hd += 8) {
    const bool isq = hd < r.heads;
    const T* src = row + (isq ? q_off + hd * r.dim : k_off + (hd - r.heads) * r.dim);
    T* dst = isq || !k_cache ? const_cast<T*>(src) : k_cache + slot * r.kv_heads * r.dim + (hd - r.heads) * r.dim;
    const float* w = isq ? r.q_norm : r.k_norm;
    float inv = 1.f;
    if (w) {
      float ss = 0.f;
      for (int d = lane; d < r.dim; d += 32) { const float x = to_f(src[d]); ss += x * x; }
      inv = 1.f / sqrtf(warp_sum(ss) / (float)r.dim + r.eps);
    }
    for (int j = lane; j < half; j += 32) {
      const int a = j * step, c = a + first;
      float u = to_f(src[a]), v = to_f(src[c]);
      if (w) { u = u * inv * w[a]; v = v * inv * w[c]; }
      dst[a] = from_f<T>(u * cs[j] - v * cs[half + j]);
      dst[c] = from_f<T>(v * cs[j] + u * cs[half + j]);
    }
    for (int d = r.rot + lane; d < r.dim; d += 32) dst[d] = w ? from_f<T>(to_f(src[d]) * inv * w[d]) : src[d];
  }
  if (k_cache) {
    T* vd = v_cache + slot * r.kv_heads * r.vdim;
    for (int e = threadIdx.x; e < r.kv_heads * r.vdim; e += blockDim.x) vd[e] = row[v_off + e];
  }
}

// The same for bf16 heads of up to 256 in pieces of 8: a lane holds one piece.  A CTA takes `span` tokens, whose heads its
// warps share; four heads of a warp are under way while four are worked on.  Pairs of neighbours lie in one lane; the other
// layout's partners are fetched from the lane half / 8 away.
__device__ __forceinline__ void unpack8(uint4 v, float (&x)[8]) {
  const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) { x[2 * i] = __uint_as_float(w[i] << 16); x[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u); }
}
__device__ __forceinline__ uint4 pack8(const float (&x)[8]) {
  uint32_t w[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 p = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
    w[i] = *reinterpret_cast<const uint32_t*>(&p);
  }
  return make_uint4(w[0], w[1], w[2], w[3]);
}
constexpr int kRopeSpan = 4;
template <bool NEIGHBOURS>
__global__ void __launch_bounds__(256, 4) norm_rope_vec_kernel(bf16* proj, bf16* k_cache, bf16* v_cache, const nqb200_rope r, const nqb200_batch bt,
                                                               int64_t stride, int q_off, int k_off, int v_off, int span) {
  extern __shared__ __align__(16) float cs[];  // [dim] q_norm, [dim] k_norm, [span][rot/2] cos, [span][rot/2] sin
  __shared__ size_t slot[kRopeSpan];
  const int half = r.rot / 2, cos_at = 2 * r.dim, sin_at = cos_at + span * half;
  grid_launch_dependents();
  if (r.q_norm)
    for (int e = threadIdx.x; e < r.dim; e += blockDim.x) { cs[e] = r.q_norm[e]; cs[r.dim + e] = r.k_norm[e]; }
  grid_dependency_wait();
  const int b = blockIdx.y, t0 = bt.cu[b], n = bt.cu[b + 1] - t0, first = blockIdx.x * span, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (first >= n) return;
  const int tokens = min(span, n - first), heads = r.heads + r.kv_heads, items = tokens * heads;
  bf16* rows = proj + (size_t)(t0 + first) * stride;
  const bool live = lane * 8 < r.dim;
  const int piece = live ? lane * 8 : 0;
  auto token_of = [&](int it) { return (it >= heads) + (it >= 2 * heads) + (it >= 3 * heads); };
  auto place = [&](int tk, int hd) { return rows + (size_t)tk * stride + (hd < r.heads ? q_off + hd * r.dim : k_off + (hd - r.heads) * r.dim) + piece; };
  constexpr int U = 4;
  uint4 in[U], next[U];
  auto request = [&](int i0, uint4 (&v)[U]) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int it = min(i0 + 8 * u, items - 1), tk = token_of(it);
      v[u] = *reinterpret_cast<const uint4*>(place(tk, it - tk * heads));
    }
  };
  request(warp, next);
  const int p0 = bt.pos0[b] + first;
  for (int e = threadIdx.x; e < tokens * half; e += blockDim.x) {
    const int tk = e / half, f = e - tk * half;
    sincosf((float)(p0 + tk) * r.inv_freq[f], &cs[sin_at + e], &cs[cos_at + e]);
  }
  if (k_cache && (int)threadIdx.x < tokens) slot[threadIdx.x] = kv_row(bt, b, p0 + threadIdx.x);
  __syncthreads();
  const bool turns = live && lane * 8 < r.rot;
  const bool upper = !NEIGHBOURS && lane * 8 >= half;
  const int partner = NEIGHBOURS || !turns ? lane : upper ? lane - half / 8 : lane + half / 8;
  const int angle = turns ? (NEIGHBOURS ? lane * 4 : lane * 8 - (upper ? half : 0)) : 0;   // of the piece's first element
  for (int i0 = warp; i0 < items; i0 += 8 * U) {
#pragma unroll
    for (int u = 0; u < U; ++u) in[u] = next[u];
    if (i0 + 8 * U < items) request(i0 + 8 * U, next);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int it = i0 + 8 * u;
      if (it >= items) break;
      const int tk = token_of(it), hd = it - tk * heads;
      float x[8], y[8];
      unpack8(in[u], x);
      if (r.q_norm) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
        const float inv = 1.f / sqrtf(warp_sum(live ? ss : 0.f) / (float)r.dim + r.eps);
        const float4* w = reinterpret_cast<const float4*>(cs + (hd < r.heads ? 0 : r.dim) + piece);
        const float4 w0 = w[0], w1 = w[1];
        const float wv[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = x[e] * inv * wv[e];
      }
      const float4* cp = reinterpret_cast<const float4*>(cs + cos_at + tk * half + angle);
      const float4* sp = reinterpret_cast<const float4*>(cs + sin_at + tk * half + angle);
      if (NEIGHBOURS) {
        const float4 c = turns ? cp[0] : make_float4(1.f, 1.f, 1.f, 1.f), s = turns ? sp[0] : make_float4(0.f, 0.f, 0.f, 0.f);
        const float cv[4] = {c.x, c.y, c.z, c.w}, sv[4] = {s.x, s.y, s.z, s.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          y[2 * e] = x[2 * e] * cv[e] - x[2 * e + 1] * sv[e];
          y[2 * e + 1] = x[2 * e + 1] * cv[e] + x[2 * e] * sv[e];
        }
      } else {
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const float4 c = turns ? cp[q] : make_float4(1.f, 1.f, 1.f, 1.f), s = turns ? sp[q] : make_float4(0.f, 0.f, 0.f, 0.f);
          const float cv[4] = {c.x, c.y, c.z, c.w}, sv[4] = {s.x, s.y, s.z, s.w};
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float other = __shfl_sync(0xFFFFFFFFu, x[4 * q + e], partner);
            y[4 * q + e] = x[4 * q + e] * cv[e] + other * (upper ? sv[e] : -sv[e]);
          }
        }
      }
      if (live) *reinterpret_cast<uint4*>(hd < r.heads || !k_cache ? place(tk, hd) : k_cache + (slot[tk] * r.kv_heads + (hd - r.heads)) * r.dim + piece) = pack8(y);
    }
  }
  if (k_cache) {
    const int per = r.kv_heads * r.vdim / 8;
    for (int e = threadIdx.x; e < tokens * per; e += blockDim.x) {
      const int tk = e / per, c = e - tk * per;
      reinterpret_cast<uint4*>(v_cache + slot[tk] * r.kv_heads * r.vdim)[c] = reinterpret_cast<const uint4*>(rows + (size_t)tk * stride + v_off)[c];
    }
  }
}

constexpr int kSimpleKeys = 128;   // keys per pass = threads
constexpr int kSimpleVCols = 8;    // value columns per thread at most: vdim <= 1024

// One CTA per (token, head): a thread scores one key per pass, then owns value columns.
template <typename T>
__global__ void __launch_bounds__(kSimpleKeys) attention_simple_kernel(const T* __restrict__ q, int64_t q_stride, const T* __restrict__ k_cache,
                                                                       const T* __restrict__ v_cache, T* __restrict__ out, int64_t out_stride,
                                                                       const nqb200_attention at, const nqb200_batch bt) {
  extern __shared__ float qs[];  // [dim]
  __shared__ float sc[kSimpleKeys];
  __shared__ int rows[kSimpleKeys];
  __shared__ float red[4];
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.z, h = blockIdx.y, i = blockIdx.x, tid = threadIdx.x, t0 = bt.cu[b];
  if (i >= bt.cu[b + 1] - t0) return;
  const int p = bt.pos0[b] + i, lo = at.chunk > 0 ? p / at.chunk * at.chunk : 0, g = h / (at.heads / at.kv_heads);
  const T* qr = q + (size_t)(t0 + i) * q_stride + (size_t)h * at.dim;
  for (int d = tid; d < at.dim; d += kSimpleKeys) qs[d] = to_f(qr[d]);
  float m = at.sink ? at.sink[h] : -INFINITY, l = at.sink ? 1.f : 0.f;
  const float factor = at.scale * (at.temp ? at.temp[h] : 1.f), shift = at.bias ? at.bias[h] : 0.f;
  float acc[kSimpleVCols] = {};
  for (int j0 = lo; j0 <= p; j0 += kSimpleKeys) {
    const int j = j0 + tid;
    __syncthreads();
    float s = -INFINITY;
    if (j <= p) {
      const size_t r = kv_row(bt, b, j);
      rows[tid] = (int)r;
      const T* kr = k_cache + (r * at.kv_heads + g) * at.dim;
      float d = 0.f;
      for (int c = 0; c < at.dim; ++c) d += qs[c] * to_f(kr[c]);
      s = d * factor + shift;
      if (at.softcap > 0.f) s = at.softcap * tanhf(s / at.softcap);
    }
    float corr = 1.f;
    if (at.sigmoid) {
      sc[tid] = sigmoid_f(s);
      __syncthreads();
    } else {
      const float wm = warp_max(s);
      if ((tid & 31) == 0) red[tid >> 5] = wm;
      __syncthreads();
      const float m_new = fmaxf(m, fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])));
      const float e = expf(s - m_new);
      corr = expf(m - m_new);
      sc[tid] = e;
      const float ws = warp_sum(e);
      __syncthreads();
      if ((tid & 31) == 0) red[tid >> 5] = ws;
      __syncthreads();
      l = l * corr + (red[0] + red[1] + red[2] + red[3]);
      m = m_new;
    }
    const int cnt = min(kSimpleKeys, p - j0 + 1);
#pragma unroll
    for (int c = 0; c < kSimpleVCols; ++c) {
      const int col = tid + c * kSimpleKeys;
      if (col >= at.vdim) break;
      float a = acc[c] * corr;
      for (int jj = 0; jj < cnt; ++jj) a += sc[jj] * to_f(v_cache[((size_t)rows[jj] * at.kv_heads + g) * at.vdim + col]);
      acc[c] = a;
    }
  }
  const float f = at.sigmoid ? at.out_scale : at.out_scale / l;
#pragma unroll
  for (int c = 0; c < kSimpleVCols; ++c) {
    const int col = tid + c * kSimpleKeys;
    if (col < at.vdim) out[(size_t)(t0 + i) * out_stride + (size_t)h * at.vdim + col] = from_f<T>(acc[c] * f);
  }
}

}  // namespace nqb200

using namespace nqb200;

extern "C" int nqb200_rope_store(void* proj, void* k_cache, void* v_cache, const float* inv_freq, const nqb200_batch* b, int64_t stride,
                                 int64_t q_off, int64_t k_off, int64_t v_off, int64_t heads, int64_t kv_heads, int64_t dim, int64_t vdim,
                                 int64_t rot, int dtype, void* stream) {
  const int st = check_batch(b, true);
  if (st != NQB200_OK) return st;
  if (heads <= 0 || kv_heads <= 0 || dim <= 0 || vdim <= 0 || rot < 0 || rot > dim || rot % 2 != 0 || stride <= 0) return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (b->tokens == 0) return NQB200_OK;
  if (!proj || !k_cache || !v_cache || (rot > 0 && !inv_freq)) return NQB200_ERR_NULL_POINTER;
  const dim3 grid((unsigned)b->max_len, (unsigned)b->batch), block(256);
  const size_t smem = (size_t)rot * sizeof(float);
#define NQB200_ROPE(T)                                                                                                                   \
  launch_overlapped(rope_store_kernel<T>, grid, block, smem, (cudaStream_t)stream, (T*)proj, (T*)k_cache, (T*)v_cache, inv_freq, *b,     \
                    (int)stride, (int)q_off, (int)k_off, (int)v_off, (int)heads, (int)kv_heads, (int)dim, (int)vdim, (int)rot)
  return dtype == NQB200_F32 ? NQB200_ROPE(float) : NQB200_ROPE(bf16);
#undef NQB200_ROPE
}

extern "C" int nqb200_norm_rope(void* proj, void* k_cache, void* v_cache, const nqb200_rope* r, const nqb200_batch* b, int64_t stride,
                                int64_t q_off, int64_t k_off, int64_t v_off, int dtype, void* stream) {
  const int st = check_batch(b, k_cache != nullptr);
  if (st != NQB200_OK) return st;
  if (!r) return NQB200_ERR_NULL_POINTER;
  if (r->heads <= 0 || r->kv_heads <= 0 || r->dim <= 0 || r->rot < 0 || r->rot > r->dim || r->rot % 2 != 0 || stride <= 0 || r->rot > 8192 ||
      (k_cache && r->vdim <= 0))
    return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (b->tokens == 0) return NQB200_OK;
  if (!proj || (k_cache && !v_cache) || (r->rot > 0 && !r->inv_freq)) return NQB200_ERR_NULL_POINTER;
  const dim3 grid((unsigned)b->max_len, (unsigned)b->batch), block(256);
  const size_t smem = (size_t)r->rot * sizeof(float);
  cudaStream_t s = (cudaStream_t)stream;
  const bool pieces = dtype == NQB200_BF16 && r->dim % 8 == 0 && r->dim <= 256 && r->rot % (r->interleaved ? 8 : 16) == 0 && stride % 8 == 0 && q_off % 8 == 0 &&
                      k_off % 8 == 0 && aligned16(proj) && (!r->q_norm || r->k_norm) && (r->q_norm || !r->k_norm) &&
                      (!k_cache || (aligned16(k_cache) && aligned16(v_cache) && r->vdim % 8 == 0 && v_off % 8 == 0));
  if (pieces) {
    auto kernel = r->interleaved ? norm_rope_vec_kernel<true> : norm_rope_vec_kernel<false>;
    const int span = b->max_len >= 4 * kNumSMs ? kRopeSpan : 1;
    return launch_overlapped(kernel, dim3((unsigned)((b->max_len + span - 1) / span), (unsigned)b->batch), block, (size_t)(2 * r->dim + span * r->rot) * sizeof(float), s,
                             (bf16*)proj, (bf16*)k_cache, (bf16*)v_cache, *r, *b, stride, (int)q_off, (int)k_off, (int)v_off, span);
  }
  if (dtype == NQB200_F32)
    return launch_overlapped(norm_rope_kernel<float>, grid, block, smem, s, (float*)proj, (float*)k_cache, (float*)v_cache, *r, *b, stride,
                             (int)q_off, (int)k_off, (int)v_off);
  return launch_overlapped(norm_rope_kernel<bf16>, grid, block, smem, s, (bf16*)proj, (bf16*)k_cache, (bf16*)v_cache, *r, *b, stride, (int)q_off,
                           (int)k_off, (int)v_off);
}

extern "C" int nqb200_chunk_attention(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, void* out,
                                      int64_t out_stride, int64_t cache_rows, const nqb200_attention* a, const nqb200_batch* b, int* status,
                                      int dtype, void* stream) {
  const int st = check_batch(b, true);
  if (st != NQB200_OK) return st;
  if (!a) return NQB200_ERR_NULL_POINTER;
  if (a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads != 0 || a->dim <= 0 || a->dim > 4096 || a->vdim <= 0 ||
      a->vdim > kSimpleKeys * kSimpleVCols || a->heads > 65535 || (a->sigmoid && (a->softcap > 0.f || a->sink)) ||
      (!a->sigmoid && (a->temp || a->bias)))
    return NQB200_ERR_BAD_SHAPE;
  if (!mixer_dtype(dtype)) return NQB200_ERR_BAD_DTYPE;
  if (b->tokens == 0) return NQB200_OK;
  if (!q || !k_cache || !v_cache || !out) return NQB200_ERR_NULL_POINTER;
  if (dtype == NQB200_BF16 && attention_umma_supports(q, q_stride, k_cache, v_cache, out, out_stride, cache_rows, a, b))
    return attention_umma(q, q_stride, k_cache, v_cache, out, out_stride, cache_rows, a, b, status, (cudaStream_t)stream);
  if (dtype == NQB200_BF16 && b->max_len > 1 && attention_prefill_supports(q, q_stride, k_cache, v_cache, out, out_stride, a))
    return attention_prefill(q, q_stride, k_cache, v_cache, out, out_stride, a, b, (cudaStream_t)stream);
  const dim3 grid((unsigned)b->max_len, (unsigned)a->heads, (unsigned)b->batch), block(kSimpleKeys);
  const size_t smem = (size_t)a->dim * sizeof(float);
#define NQB200_ATT(T)                                                                                                              \
  launch_overlapped(attention_simple_kernel<T>, grid, block, smem, (cudaStream_t)stream, (const T*)q, q_stride, (const T*)k_cache, \
                    (const T*)v_cache, (T*)out, out_stride, *a, *b)
  return dtype == NQB200_F32 ? NQB200_ATT(float) : NQB200_ATT(bf16);
#undef NQB200_ATT
}
