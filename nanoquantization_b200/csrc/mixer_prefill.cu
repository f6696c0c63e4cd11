// Tensor-core kernels (bf16) for prompts and portions of prompts: chunk-masked attention over the paged cache, and
// retention in chunkwise form.
//
// One CTA takes 128 query tokens of one head: 8 warps of 16 rows, key tiles of 64 through a two-stage cp.async ring,
// mma.m16n8k16 with float accumulators, scores and weights in float.  Both mixers share the loop.  Attention: scaled,
// capped scores, online softmax that starts from the sink; or sigmoid weights, summed as they are.  Retention: keys are those of the query's own chunk of 256
// tokens (counted from the step's first token), a score is weighted by decay^(i-j), and what lies before the chunk
// comes as decay^(i+1) q S with S the state at the chunk's start; the head's norm and gate close the row.
//
// The states at the chunk starts come from two kernels ahead: the chunks' own contributions sum_j decay^(len-1-j) k_j
// v_j^T, all in parallel, then a scan over the chunks.  Where a float value has to be a tensor-core operand there
// (a state, a weighted v) it is split into two bf16 numbers, so that states keep about 16 bits through every product.
#include "mixers.cuh"
#include "mma_utils.cuh"

namespace nqb200 {

constexpr int kRows = 128, kKeys = 64, kThreads = 256;
constexpr int kRetChunk = 256;

// tanh to within a few float ulps of 1: 1 - 2 / (1 + e^2y), right at both ends.
__device__ __forceinline__ float tanh_exp(float y) { return 1.f - __fdividef(2.f, 1.f + exp2f(y * 2.885390082f)); }
// decay^n for n >= 0
__device__ __forceinline__ float decay_pow(float log2d, int n) { return n == 0 ? 1.f : exp2f((float)n * log2d); }

struct PrefillArgs {
  const bf16* q; int64_t q_stride;          // head h at column h * dim
  bf16* out; int64_t out_stride;            // head h at column h * vdim
  nqb200_batch bt;
  int heads, dim, vdim;
  float out_scale;
  // attention
  const bf16* k_cache; const bf16* v_cache;
  int kv_heads, chunk;
  float scale, softcap;
  const float* sink;
  int sigmoid; const float* temp; const float* bias;
  // retention: k, v, gate in the same buffer as q
  const bf16* k; const bf16* v; const bf16* gate;
  const float* decay; const bf16* states;    // states [chunk id][heads][high part, rest][dim][vdim]
  float eps; const float* norm;
};

// Chunk c of sequence b has id cu[b] / 256 + b + c: distinct, and below tokens / 256 + batch.
__device__ __forceinline__ size_t chunk_id(const nqb200_batch& bt, int b, int c) { return (size_t)(bt.cu[b] / kRetChunk + b + c); }

template <int DP, int VP, bool RET>
__global__ void __launch_bounds__(kThreads, 1) prefill_kernel(const PrefillArgs a) {
  constexpr int QS = DP + 8, VS = VP + 8;   // row strides: 16-byte chunks fall on different banks
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* qs = reinterpret_cast<bf16*>(smem_raw);
  bf16* ks = qs + kRows * QS;
  bf16* vs = ks + 2 * kKeys * QS;
  float* pw = reinterpret_cast<float*>(vs + 2 * kKeys * VS);   // [kRetChunk + 1], retention only
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int t0 = a.bt.cu[b], n = a.bt.cu[b + 1] - t0, i0 = blockIdx.x * kRows;
  if (i0 >= n) return;
  const int pos0 = RET ? 0 : a.bt.pos0[b];        // retention counts from the step's first token
  const int p0 = pos0 + i0, plast = pos0 + min(i0 + kRows, n) - 1;
  const int size = RET ? kRetChunk : a.chunk;
  const int kstart = size > 0 ? p0 / size * size : 0;
  const int D8 = a.dim / 8, V8 = a.vdim / 8;

  // zero what the copies never write: columns past dim and vdim
  for (int e = tid; e < (kRows + 2 * kKeys) * (DP - a.dim); e += kThreads) qs[(e / (DP - a.dim)) * QS + a.dim + e % (DP - a.dim)] = __float2bfloat16_rn(0.f);
  for (int e = tid; e < 2 * kKeys * (VP - a.vdim); e += kThreads) vs[(e / (VP - a.vdim)) * VS + a.vdim + e % (VP - a.vdim)] = __float2bfloat16_rn(0.f);
  for (int e = tid; e < kRows * D8; e += kThreads) {
    const int r = e / D8, c = e % D8;
    const bool ok = i0 + r < n;
    cp16(smem_addr(qs + r * QS + c * 8), a.q + (size_t)(t0 + (ok ? i0 + r : i0)) * a.q_stride + (size_t)h * a.dim + c * 8, ok);
  }
  const int kvh = RET ? h : h / (a.heads / a.kv_heads);
  auto load_tile = [&](int j0, int stage) {   // keys j0 .. j0 + 63: four threads per key
    const int key = tid >> 2, j = j0 + key;
    const bool ok = j <= plast;
    const bf16 *kp, *vp;
    if (RET) {
      const size_t row = (size_t)(t0 + (ok ? j : i0)) * a.q_stride;
      kp = a.k + row + (size_t)h * a.dim;
      vp = a.v + row + (size_t)h * a.vdim;
    } else {
      const size_t row = (kv_row(a.bt, b, ok ? j : p0) * a.kv_heads + kvh);
      kp = a.k_cache + row * a.dim;
      vp = a.v_cache + row * a.vdim;
    }
    bf16* kd = ks + (stage * kKeys + key) * QS;
    bf16* vd = vs + (stage * kKeys + key) * VS;
    for (int c = tid & 3; c < D8; c += 4) cp16(smem_addr(kd + c * 8), kp + c * 8, ok);
    for (int c = tid & 3; c < V8; c += 4) cp16(smem_addr(vd + c * 8), vp + c * 8, ok);
  };

  float O[VP / 8][4];
#pragma unroll
  for (int i = 0; i < VP / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) O[i][e] = 0.f;
  const int w0 = p0 + warp * 16, wlast = min(w0 + 15, plast);      // this warp's query positions
  const int pr[2] = {w0 + g, w0 + g + 8};
  int lor[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) lor[r] = size > 0 ? pr[r] / size * size : 0;
  float m[2], l[2];
  const float sink = (!RET && a.sink) ? a.sink[h] : -INFINITY;
#pragma unroll
  for (int r = 0; r < 2; ++r) { m[r] = sink; l[r] = (!RET && a.sink && t == 0) ? 1.f : 0.f; }
  const bf16* qw = qs + warp * 16 * QS;
  const uint32_t q_addr = smem_addr(qw + (lane & 15) * QS + (lane >> 4) * 8);
  const uint32_t k_lane = ((lane & 7) + ((lane >> 4) << 3)) * QS + ((lane >> 3) & 1) * 8;
  const uint32_t v_lane = ((lane & 7) + (((lane >> 3) & 1) << 3)) * VS + (lane >> 4) * 8;
  const float log2d = RET ? log2f(a.decay[h]) : 0.f;
  const float factor = !RET && a.temp ? a.scale * a.temp[h] : a.scale, shift = !RET && a.bias ? a.bias[h] : 0.f;

  if (RET) {
    for (int e = tid; e <= kRetChunk; e += kThreads) pw[e] = decay_pow(log2d, e);
    cp_commit();
    cp_wait<0>();
    __syncthreads();
    // the part from before this chunk: q S, then rows times decay^(i + 1)
    const bf16* S = a.states + (chunk_id(a.bt, b, kstart / kRetChunk) * a.heads + h) * (size_t)(2 * a.dim * a.vdim);
    for (int d0 = 0; d0 < DP; d0 += kKeys) {
      __syncthreads();
      const int r = tid >> 2;             // four threads per row, both parts
      const bool ok = d0 + r < a.dim;
      const bf16* src = S + (size_t)(ok ? d0 + r : 0) * a.vdim;
      for (int c = tid & 3; c < V8; c += 4) {
        cp16(smem_addr(vs + r * VS + c * 8), src + c * 8, ok);
        cp16(smem_addr(vs + (kKeys + r) * VS + c * 8), src + (size_t)a.dim * a.vdim + c * 8, ok);
      }
      cp_commit();
      cp_wait<0>();
      __syncthreads();
#pragma unroll
      for (int kt = 0; kt < kKeys / 16; ++kt) {
        if (d0 + kt * 16 >= DP) break;
        uint32_t qa[4];
        ldsm4(qa, q_addr + (d0 + kt * 16) * 2);
#pragma unroll
        for (int part = 0; part < 2; ++part) {
          const uint32_t base = smem_addr(vs + (part * kKeys + kt * 16) * VS) + v_lane * 2;
#pragma unroll
          for (int nt = 0; nt < VP / 16; ++nt) {
            uint32_t vb[4];
            ldsm4t(vb, base + nt * 32);
            mma(O[2 * nt], qa, vb[0], vb[1]);
            mma(O[2 * nt + 1], qa, vb[2], vb[3]);
          }
        }
      }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const float f = pw[min(pr[r] - kstart + 1, kRetChunk)];
#pragma unroll
      for (int i = 0; i < VP / 8; ++i) { O[i][2 * r] *= f; O[i][2 * r + 1] *= f; }
    }
    __syncthreads();
  }

  load_tile(kstart, 0);
  cp_commit();
  int stage = 0;
  for (int j0 = kstart; j0 <= plast; j0 += kKeys, stage ^= 1) {
    const bool more = j0 + kKeys <= plast;
    if (more) load_tile(j0 + kKeys, stage ^ 1);
    cp_commit();
    cp_wait<1>();
    __syncthreads();
    const int wlo = size > 0 ? w0 / size * size : 0;
    if (w0 <= plast && j0 <= wlast && j0 + kKeys > wlo) {
      float s[kKeys / 8][4];
#pragma unroll
      for (int i = 0; i < kKeys / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
      const uint32_t kb = smem_addr(ks + stage * kKeys * QS) + k_lane * 2;
#pragma unroll
      for (int kt = 0; kt < DP / 16; ++kt) {
        uint32_t qa[4];
        ldsm4(qa, q_addr + kt * 32);
#pragma unroll
        for (int nt = 0; nt < kKeys / 16; ++nt) {
          uint32_t kf[4];
          ldsm4(kf, kb + (nt * 16 * QS + kt * 16) * 2);
          mma(s[2 * nt], qa, kf[0], kf[1]);
          mma(s[2 * nt + 1], qa, kf[2], kf[3]);
        }
      }
      const int wlasto = size > 0 ? wlast / size * size : 0;
      const bool mask = j0 + kKeys - 1 > w0 || j0 < wlasto;
      if (RET) {
        const float ksc = a.scale;
#pragma unroll
        for (int i = 0; i < kKeys / 8; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int j = j0 + i * 8 + 2 * t + (e & 1), dist = pr[e >> 1] - j;
            s[i][e] = (dist >= 0 && j >= lor[e >> 1]) ? s[i][e] * (ksc * pw[min(dist, kRetChunk)]) : 0.f;
          }
      } else if (a.sigmoid) {
#pragma unroll
        for (int i = 0; i < kKeys / 8; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int j = j0 + i * 8 + 2 * t + (e & 1);
            const float w = sigmoid_fast(s[i][e] * factor + shift);
            s[i][e] = (mask && (j > pr[e >> 1] || j < lor[e >> 1])) ? 0.f : w;
          }
      } else {
        float mx[2] = {m[0], m[1]};
#pragma unroll
        for (int i = 0; i < kKeys / 8; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float v = s[i][e] * a.scale;
            if (a.softcap > 0.f) v = a.softcap * tanh_exp(__fdividef(v, a.softcap));
            if (mask) {
              const int j = j0 + i * 8 + 2 * t + (e & 1);
              if (j > pr[e >> 1] || j < lor[e >> 1]) v = -INFINITY;
            }
            s[i][e] = v;
            mx[e >> 1] = fmaxf(mx[e >> 1], v);
          }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const float mn = quad_max(mx[r]), use = mn == -INFINITY ? 0.f : mn, corr = exp2f((m[r] - use) * 1.4426950409f);
          m[r] = mn;
          l[r] *= corr;
#pragma unroll
          for (int i = 0; i < VP / 8; ++i) { O[i][2 * r] *= corr; O[i][2 * r + 1] *= corr; }
#pragma unroll
          for (int i = 0; i < kKeys / 8; ++i)
#pragma unroll
            for (int e = 2 * r; e < 2 * r + 2; ++e) {
              s[i][e] = exp2f((s[i][e] - use) * 1.4426950409f);
              l[r] += s[i][e];
            }
        }
      }
#pragma unroll
      for (int kt = 0; kt < kKeys / 16; ++kt) {
        const uint32_t pa[4] = {pack2(s[2 * kt][0], s[2 * kt][1]), pack2(s[2 * kt][2], s[2 * kt][3]), pack2(s[2 * kt + 1][0], s[2 * kt + 1][1]),
                                pack2(s[2 * kt + 1][2], s[2 * kt + 1][3])};
        const uint32_t base = smem_addr(vs + (stage * kKeys + kt * 16) * VS) + v_lane * 2;
#pragma unroll
        for (int nt = 0; nt < VP / 16; ++nt) {
          uint32_t vb[4];
          ldsm4t(vb, base + nt * 32);
          mma(O[2 * nt], pa, vb[0], vb[1]);
          mma(O[2 * nt + 1], pa, vb[2], vb[3]);
        }
      }
    }
    __syncthreads();
  }
  cp_wait<0>();

#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float f;
    if (RET) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < VP / 8; ++i) ss += O[i][2 * r] * O[i][2 * r] + O[i][2 * r + 1] * O[i][2 * r + 1];
      f = a.out_scale / sqrtf(quad_sum(ss) / (float)a.vdim + a.eps);
    } else {
      const float sum = quad_sum(l[r]);
      f = a.sigmoid ? a.out_scale : a.out_scale / sum;
    }
    if (pr[r] > plast) continue;
    const size_t tok = (size_t)(t0 + pr[r] - pos0);
    bf16* dst = a.out + tok * a.out_stride + (size_t)h * a.vdim;
    const bf16* gp = RET ? a.gate + tok * a.q_stride + (size_t)h * a.vdim : nullptr;
    constexpr int U = VP / 8 < 16 ? VP / 8 : 16;   // loads under way at once (from places that exist)
#pragma unroll
    for (int i1 = 0; i1 < VP / 8; i1 += U) {
      uint32_t gw[U];
      float2 nw[U];
      if (RET) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int c = (i1 + u) * 8 + 2 * t, cc = c < a.vdim ? c : 0;
          gw[u] = *reinterpret_cast<const uint32_t*>(gp + cc);
          nw[u] = a.norm ? *reinterpret_cast<const float2*>(a.norm + cc) : make_float2(1.f, 1.f);
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = i1 + u, c = i * 8 + 2 * t;
        float x = O[i][2 * r] * f, y = O[i][2 * r + 1] * f;
        if (RET) {
          const float gx = __uint_as_float(gw[u] << 16), gy = __uint_as_float(gw[u] & 0xFFFF0000u);
          x *= nw[u].x * (gx * sigmoid_fast(gx));
          y *= nw[u].y * (gy * sigmoid_fast(gy));
        }
        if (c < a.vdim) *reinterpret_cast<uint32_t*>(dst + c) = pack2(x, y);
      }
    }
  }
}

// Contribution of one chunk to the state, a tile of 64 x 64 of (dim x vdim) per CTA.
struct ChunkStateArgs {
  const bf16* k; const bf16* v; int64_t stride;
  const float* decay; float* states;
  int heads, dim, vdim, vtiles;
  nqb200_batch bt;
};
constexpr int kTS = 64 + 8;
__global__ void __launch_bounds__(128) retention_chunk_kernel(const ChunkStateArgs a) {
  __shared__ __align__(16) bf16 ks[64 * kTS], vh[64 * kTS], vl[64 * kTS];
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.z, c = blockIdx.x, t0 = a.bt.cu[b], n = a.bt.cu[b + 1] - t0, first = c * kRetChunk;
  if (first >= n) return;
  const int tiles = (a.dim + 63) / 64 * a.vtiles, h = blockIdx.y / tiles, tile = blockIdx.y % tiles;
  const int d0 = tile / a.vtiles * 64, v0 = tile % a.vtiles * 64, len = min(kRetChunk, n - first);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const float log2d = log2f(a.decay[h]), kscale = 1.f / sqrtf((float)a.dim);
  float acc[8][4] = {};
  const uint32_t a_addr = smem_addr(ks + ((lane & 7) + ((lane >> 4) << 3)) * kTS + warp * 16 + ((lane >> 3) & 1) * 8);
  const uint32_t b_lane = (((lane & 7) + (((lane >> 3) & 1) << 3)) * kTS + (lane >> 4) * 8) * 2;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  // a thread's 16-byte pieces: rows tid / 8 + 16 i of the tile, loaded a tile ahead (from places that exist) into registers
  const int r0 = tid >> 3, cc = (tid & 7) * 8, kcol = min(d0 + cc, a.dim - 8), vcol = min(v0 + cc, a.vdim - 8);
  uint4 kreg[4], vreg[4];
  auto fetch = [&](int j0) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const size_t row = (size_t)(t0 + first + min(j0 + r0 + 16 * i, len - 1)) * a.stride;
      kreg[i] = *reinterpret_cast<const uint4*>(a.k + row + (size_t)h * a.dim + kcol);
      vreg[i] = *reinterpret_cast<const uint4*>(a.v + row + (size_t)h * a.vdim + vcol);
    }
  };
  fetch(0);
  for (int j0 = 0; j0 < len; j0 += 64) {
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = r0 + 16 * i, j = j0 + r;
      const uint4 kv = d0 + cc < a.dim ? kreg[i] : zero, vv = v0 + cc < a.vdim ? vreg[i] : zero;
      *reinterpret_cast<uint4*>(ks + r * kTS + cc) = kv;
      const float w = j < len ? kscale * decay_pow(log2d, len - 1 - j) : 0.f;
      const uint32_t in[4] = {vv.x, vv.y, vv.z, vv.w};
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float x = __uint_as_float(in[k] << 16) * w, y = __uint_as_float(in[k] & 0xFFFF0000u) * w;
        const float hx = __bfloat162float(__float2bfloat16_rn(x)), hy = __bfloat162float(__float2bfloat16_rn(y));
        hi[k] = pack2(hx, hy);
        lo[k] = pack2(x - hx, y - hy);
      }
      *reinterpret_cast<uint4*>(vh + r * kTS + cc) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(vl + r * kTS + cc) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    __syncthreads();
    if (j0 + 64 < len) fetch(j0 + 64);
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      uint32_t ka[4];
      ldsm4t(ka, a_addr + kt * 16 * kTS * 2);
#pragma unroll
      for (int part = 0; part < 2; ++part) {
        const uint32_t base = smem_addr((part ? vl : vh) + kt * 16 * kTS) + b_lane;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          uint32_t vb[4];
          ldsm4t(vb, base + nt * 32);
          mma(acc[2 * nt], ka, vb[0], vb[1]);
          mma(acc[2 * nt + 1], ka, vb[2], vb[3]);
        }
      }
    }
  }
  float* S = a.states + (chunk_id(a.bt, b, c) * a.heads + h) * (size_t)a.dim * a.vdim;
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int d = d0 + warp * 16 + g + 8 * r, v = v0 + i * 8 + 2 * t;
      if (d < a.dim && v < a.vdim) *reinterpret_cast<float2*>(S + (size_t)d * a.vdim + v) = make_float2(acc[i][2 * r], acc[i][2 * r + 1]);
    }
}

// starts[c] <- the state ahead of chunk c, split into two bf16 numbers; the sequence's own state moves to the end of the step.
__global__ void __launch_bounds__(256) retention_scan_kernel(const float* __restrict__ states, bf16* __restrict__ starts, float* state,
                                                             const float* __restrict__ decay, int heads, int per_head, const nqb200_batch bt) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.z, h = blockIdx.y, e = (blockIdx.x * 256 + threadIdx.x) * 4, n = bt.cu[b + 1] - bt.cu[b];
  if (e >= per_head || n <= 0) return;
  const float log2d = log2f(decay[h]);
  float* own = state + ((size_t)bt.slot[b] * heads + h) * per_head + e;
  float4 S = bt.pos0[b] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(own);
  const int chunks = (n + kRetChunk - 1) / kRetChunk;
  const float* p = states + (chunk_id(bt, b, 0) * heads + h) * (size_t)per_head + e;
  bf16* o = starts + (chunk_id(bt, b, 0) * heads + h) * (size_t)(2 * per_head) + e;
  const size_t step = (size_t)heads * per_head;
  float4 next = *reinterpret_cast<const float4*>(p);
  for (int c = 0; c < chunks; ++c, p += step, o += 2 * step) {
    const float4 dl = next;
    if (c + 1 < chunks) next = *reinterpret_cast<const float4*>(p + step);
    const float hx = __bfloat162float(__float2bfloat16_rn(S.x)), hy = __bfloat162float(__float2bfloat16_rn(S.y));
    const float hz = __bfloat162float(__float2bfloat16_rn(S.z)), hw = __bfloat162float(__float2bfloat16_rn(S.w));
    *reinterpret_cast<uint2*>(o) = make_uint2(pack2(hx, hy), pack2(hz, hw));
    *reinterpret_cast<uint2*>(o + per_head) = make_uint2(pack2(S.x - hx, S.y - hy), pack2(S.z - hz, S.w - hw));
    const float f = decay_pow(log2d, min(kRetChunk, n - c * kRetChunk));
    S.x = f * S.x + dl.x; S.y = f * S.y + dl.y; S.z = f * S.z + dl.z; S.w = f * S.w + dl.w;
  }
  *reinterpret_cast<float4*>(own) = S;
}

template <int DP, int VP, bool RET>
static int launch_prefill(const PrefillArgs& a, cudaStream_t st) {
  const size_t smem = ((size_t)(kRows + 2 * kKeys) * (DP + 8) + (size_t)2 * kKeys * (VP + 8)) * sizeof(bf16) + (RET ? (kRetChunk + 1) * sizeof(float) : 0);
  if (cudaFuncSetAttribute(prefill_kernel<DP, VP, RET>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return NQB200_ERR_LAUNCH;
  }
  const dim3 grid((unsigned)((a.bt.max_len + kRows - 1) / kRows), (unsigned)a.heads, (unsigned)a.bt.batch);
  return launch_overlapped(prefill_kernel<DP, VP, RET>, grid, dim3(kThreads), smem, st, a);
}
template <bool RET>
static int dispatch_prefill(const PrefillArgs& a, cudaStream_t st) {
#define NQB200_PF(D, V) return launch_prefill<D, V, RET>(a, st)
#define NQB200_PFV(D)                   \
  do {                                  \
    if (a.vdim <= 64) NQB200_PF(D, 64); \
    if (a.vdim <= 128) NQB200_PF(D, 128); \
    NQB200_PF(D, 256);                  \
  } while (0)
  if (a.dim <= 64) NQB200_PFV(64);
  if (a.dim <= 128) NQB200_PFV(128);
  NQB200_PFV(256);
#undef NQB200_PFV
#undef NQB200_PF
}

static bool prefill_sizes(int64_t heads, int64_t dim, int64_t vdim, int64_t stride, const void* p) {
  return heads > 0 && heads <= 65535 && dim > 0 && dim % 8 == 0 && dim <= 256 && vdim > 0 && vdim % 8 == 0 && vdim <= 256 && stride % 8 == 0 && aligned16(p);
}

// Called by nqb200_chunk_attention for bf16; false: the sizes or alignments are not the tensor-core kernel's.
bool attention_prefill_supports(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, const void* out, int64_t out_stride,
                                const nqb200_attention* a) {
  return prefill_sizes(a->heads, a->dim, a->vdim, q_stride, q) && aligned16(k_cache) && aligned16(v_cache) && out_stride % 2 == 0 &&
         (reinterpret_cast<uintptr_t>(out) & 3) == 0;
}
int attention_prefill(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, void* out, int64_t out_stride,
                      const nqb200_attention* a, const nqb200_batch* b, cudaStream_t st) {
  PrefillArgs p = {};
  p.q = (const bf16*)q; p.q_stride = q_stride; p.out = (bf16*)out; p.out_stride = out_stride; p.bt = *b;
  p.heads = a->heads; p.dim = a->dim; p.vdim = a->vdim; p.out_scale = a->out_scale;
  p.k_cache = (const bf16*)k_cache; p.v_cache = (const bf16*)v_cache; p.kv_heads = a->kv_heads; p.chunk = a->chunk;
  p.scale = a->scale; p.softcap = a->softcap; p.sink = a->sink; p.sigmoid = a->sigmoid; p.temp = a->temp; p.bias = a->bias;
  return dispatch_prefill<false>(p, st);
}

}  // namespace nqb200

using namespace nqb200;

extern "C" int64_t nqb200_retention_chunks(int64_t tokens, int64_t batch) { return tokens / kRetChunk + batch; }

extern "C" int nqb200_retention_prefill_supported(const nqb200_retention_desc* r, int64_t stride, int64_t off, int64_t act_stride, int64_t act_col) {
  return r && r->rank <= 0 && r->heads > 0 && r->dim > 0 && r->dim % 8 == 0 && r->dim <= 256 && r->vdim > 0 && r->vdim % 8 == 0 && r->vdim <= 256 &&
                 (int64_t)r->heads * ((r->dim + 63) / 64) * ((r->vdim + 63) / 64) <= 65535 && stride % 8 == 0 && off % 8 == 0 && act_stride % 2 == 0 &&
                 act_col % 2 == 0
             ? 1
             : 0;
}

extern "C" int nqb200_retention_prefill(const void* proj, int64_t stride, int64_t off, void* act, int64_t act_stride, int64_t act_col,
                                        const nqb200_retention_desc* r, float* state, float* chunk_states, const nqb200_batch* b, void* stream) {
  const int s = check_batch(b, false);
  if (s != NQB200_OK) return s;
  if (!nqb200_retention_prefill_supported(r, stride, off, act_stride, act_col)) return NQB200_ERR_BAD_SHAPE;
  if (b->tokens == 0) return NQB200_OK;
  if (!proj || !act || !state || !chunk_states || !r->decay) return NQB200_ERR_NULL_POINTER;
  if (!aligned16(proj) || !aligned16(act) || !aligned16(state) || !aligned16(chunk_states)) return NQB200_ERR_MISALIGNED;
  cudaStream_t st = (cudaStream_t)stream;
  const bf16* q = (const bf16*)proj + off;
  const int64_t qk = (int64_t)r->heads * r->dim, vv = (int64_t)r->heads * r->vdim;
  const unsigned chunks = (unsigned)((b->max_len + kRetChunk - 1) / kRetChunk);
  ChunkStateArgs c = {};
  c.k = q + qk; c.v = q + 2 * qk; c.stride = stride; c.decay = r->decay; c.states = chunk_states;
  c.heads = r->heads; c.dim = r->dim; c.vdim = r->vdim; c.vtiles = (r->vdim + 63) / 64; c.bt = *b;
  int rc = launch_overlapped(retention_chunk_kernel, dim3(chunks, (unsigned)(r->heads * ((r->dim + 63) / 64) * c.vtiles), (unsigned)b->batch), dim3(128), 0, st, c);
  if (rc != NQB200_OK) return rc;
  const int per_head = r->dim * r->vdim;
  bf16* starts = reinterpret_cast<bf16*>(chunk_states + nqb200_retention_chunks(b->tokens, b->batch) * r->heads * per_head);
  rc = launch_overlapped(retention_scan_kernel, dim3((unsigned)((per_head / 4 + 255) / 256), (unsigned)r->heads, (unsigned)b->batch), dim3(256), 0, st,
                         (const float*)chunk_states, starts, state, r->decay, r->heads, per_head, *b);
  if (rc != NQB200_OK) return rc;
  PrefillArgs p = {};
  p.q = q; p.q_stride = stride; p.out = (bf16*)act + act_col; p.out_stride = act_stride; p.bt = *b;
  p.heads = r->heads; p.dim = r->dim; p.vdim = r->vdim; p.out_scale = r->out_scale; p.kv_heads = r->heads;
  p.k = q + qk; p.v = q + 2 * qk; p.gate = q + 2 * qk + vv;
  p.decay = r->decay; p.states = starts; p.eps = r->eps; p.norm = r->norm; p.scale = 1.f / sqrtf((float)r->dim);
  return dispatch_prefill<true>(p, st);
}
