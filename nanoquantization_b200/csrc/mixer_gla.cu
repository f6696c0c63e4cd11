// Gated linear attention of prompts (bf16) in chunkwise form, on the tensor cores.
//
// With b_i the running sum of the log decays of a key channel inside a chunk of 128 tokens, token j weighs exp(b_i - b_j)
// in what token i >= j sees.  Exponents are only ever taken of differences that are not positive (but for one case, see
// below), so nothing overflows however fast a channel forgets:
//   gla_decay_kernel   the decays and their running sums b, float.
//   gla_chunk_kernel   what a chunk adds to the state: sum_j (k_j exp(b_end - b_j)) v_j^T.  The weighted keys enter the product
//                      as two bf16 numbers each, so that states keep about 16 bits.
//   gla_scan_kernel    S <- exp(b_end) S + contribution over the chunks: the states at their starts (two bf16 numbers each),
//                      and the sequence's own state at the end of the step.
//   gla_output_kernel  a CTA per (chunk, head), a warp per 16 tokens (a block): (q_i exp(b_i)) S, plus the scores inside the
//                      chunk.  Keys are kept as k_j exp(b at the end of j's block - b_j); the queries of a block take
//                      exp(b_i - b at the end of the key's block), which is q_i exp(b_i - b at the end of the block before
//                      theirs) times a factor per channel.  Inside the block itself that factor is above one; where a
//                      channel's decays of 16 tokens multiply to less than exp(-40) the block's own scores are summed in
//                      float, pair by pair.  Head norm, its weight and the gate close the row.
#include "mixers.cuh"
#include "mma_utils.cuh"

namespace nqb200 {
namespace gla {

constexpr int kChunk = 128, kBlock = 16, kBlocks = kChunk / kBlock, kThreads = 256;
constexpr float kMaxSpan = 40.f;

struct Args {
  const bf16* proj; int64_t stride;
  int q_off, k_off, v_off, g_off, l_off;
  bf16* act; int64_t act_stride;            // from the mixer's first column
  nqb200_retention_desc r;
  float* state;
  float* cum;                               // [tokens][heads * dim] running sums of the log decays inside the chunk
  float* add;                               // [chunk id][heads][dim][vdim] contributions
  bf16* starts;                             // [chunk id][heads][high part, rest][dim][vdim]
  nqb200_batch bt;
};

// Chunk c of sequence b has id cu[b] / 128 + b + c: distinct, and below tokens / 128 + batch.
__device__ __forceinline__ size_t chunk_id(const nqb200_batch& bt, int b, int c) { return (size_t)(bt.cu[b] / kChunk + b + c); }

constexpr int kDecayChannels = 128, kDecayStep = 16;
__global__ void __launch_bounds__(kDecayChannels) gla_decay_kernel(const Args a) {
  extern __shared__ float4 low_smem[];
  float* low_s = reinterpret_cast<float*>(low_smem);   // [rank][chunk]
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.z, t0 = a.bt.cu[b], n = a.bt.cu[b + 1] - t0, first = blockIdx.y * kChunk, rank = a.r.rank;
  if (first >= n) return;
  const int len = min(kChunk, n - first), channels = a.r.heads * a.r.dim;
  for (int e = threadIdx.x; e < kChunk * rank; e += kDecayChannels)
    low_s[e % rank * kChunk + e / rank] = to_f(a.proj[(size_t)(t0 + first + min(e / rank, len - 1)) * a.stride + a.l_off + e % rank]);
  __syncthreads();
  const int c = blockIdx.x * kDecayChannels + threadIdx.x;
  if (c >= channels) return;
  const bf16* w = reinterpret_cast<const bf16*>(a.r.a2) + (size_t)c * rank;
  const float bias = a.r.a2_bias[c], inv_tau = 1.f / a.r.tau;
  float run = 0.f;
  for (int i0 = 0; i0 < len; i0 += kDecayStep) {
    float z[kDecayStep];
#pragma unroll
    for (int i = 0; i < kDecayStep; ++i) z[i] = bias;
    for (int r = 0; r < rank; ++r) {
      const float wr = to_f(w[r]);
      const float4* lr = reinterpret_cast<const float4*>(low_s + r * kChunk + i0);
#pragma unroll
      for (int i = 0; i < kDecayStep / 4; ++i) {
        const float4 l = lr[i];
        z[4 * i] += wr * l.x; z[4 * i + 1] += wr * l.y; z[4 * i + 2] += wr * l.z; z[4 * i + 3] += wr * l.w;
      }
    }
#pragma unroll
    for (int i = 0; i < kDecayStep; ++i) {
      if (i0 + i >= len) break;
      run += (fminf(z[i], 0.f) - log1pf(exp_fast(-fabsf(z[i])))) * inv_tau;
      a.cum[(size_t)(t0 + first + i0 + i) * channels + c] = run;
    }
  }
}

// A CTA: 64 key channels x up to 256 value columns of one chunk's contribution; warps 4 (16 channels) x 2 (VP / 2 columns).
template <int VP>
__global__ void __launch_bounds__(kThreads) gla_chunk_kernel(const Args a) {
  constexpr int KS = 64 + 8, VS = VP + 8, NT = VP / 16;   // n-tiles of 8 columns per warp
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* kh = reinterpret_cast<bf16*>(smem_raw);           // [64 tokens][64 channels], weighted, high parts
  bf16* kl = kh + 64 * KS;
  bf16* vs = kl + 64 * KS;                                // [64 tokens][VP]
  grid_launch_dependents();
  grid_dependency_wait();
  const int dtiles = (a.r.dim + 63) / 64, b = blockIdx.z, h = blockIdx.y / dtiles, d0 = blockIdx.y % dtiles * 64;
  const int t0 = a.bt.cu[b], n = a.bt.cu[b + 1] - t0, first = blockIdx.x * kChunk;
  if (first >= n) return;
  const int len = min(kChunk, n - first), D = a.r.dim, V = a.r.vdim, channels = a.r.heads * D, V8 = V / 8;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3, wd = warp & 3, wv = warp >> 2;
  const float kscale = 1.f / sqrtf((float)D);
  const float* cum = a.cum + (size_t)(t0 + first) * channels + h * D;
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  const uint32_t a_off = (((lane & 7) + ((lane >> 4) << 3)) * KS + wd * 16 + ((lane >> 3) & 1) * 8) * 2;
  const uint32_t b_addr = smem_addr(vs) + (((lane & 7) + (((lane >> 3) & 1) << 3)) * VS + wv * (VP / 2) + (lane >> 4) * 8) * 2;
  // a thread weighs two neighbouring channels of 8 tokens
  const int c2 = (tid & 31) * 2, r0 = tid >> 5;
  const bool live = d0 + c2 < D;
  float2 last = make_float2(0.f, 0.f);
  if (live) last = *reinterpret_cast<const float2*>(cum + (size_t)(len - 1) * channels + d0 + c2);
  for (int j0 = 0; j0 < len; j0 += 64) {
    __syncthreads();
    for (int e = tid; e < 64 * (VP / 8); e += kThreads) {   // columns past V become zeros
      const int r = e / (VP / 8), c = e % (VP / 8);
      const bool ok = j0 + r < len && c < V8;
      cp16(smem_addr(vs + r * VS + c * 8), a.proj + (size_t)(t0 + first + (ok ? j0 + r : 0)) * a.stride + a.v_off + (size_t)h * V + (ok ? c * 8 : 0), ok);
    }
    cp_commit();
    float2 bb[8];
    uint32_t kk[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {   // all loads under way at once, from places that exist
      const int j = min(j0 + r0 + 8 * i, len - 1), c = live ? d0 + c2 : 0;
      bb[i] = *reinterpret_cast<const float2*>(cum + (size_t)j * channels + c);
      kk[i] = *reinterpret_cast<const uint32_t*>(a.proj + (size_t)(t0 + first + j) * a.stride + a.k_off + (size_t)h * D + c);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const bool ok = live && j0 + r0 + 8 * i < len;
      const float x = ok ? __uint_as_float(kk[i] << 16) * kscale * exp_fast(last.x - bb[i].x) : 0.f;
      const float y = ok ? __uint_as_float(kk[i] & 0xFFFF0000u) * kscale * exp_fast(last.y - bb[i].y) : 0.f;
      const float hx = __bfloat162float(__float2bfloat16_rn(x)), hy = __bfloat162float(__float2bfloat16_rn(y));
      *reinterpret_cast<uint32_t*>(kh + (r0 + 8 * i) * KS + c2) = pack2(hx, hy);
      *reinterpret_cast<uint32_t*>(kl + (r0 + 8 * i) * KS + c2) = pack2(x - hx, y - hy);
    }
    cp_wait<0>();
    __syncthreads();
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      uint32_t ah[4], al[4];
      ldsm4t(ah, smem_addr(kh) + a_off + kt * 16 * KS * 2);
      ldsm4t(al, smem_addr(kl) + a_off + kt * 16 * KS * 2);
#pragma unroll
      for (int nt = 0; nt < NT / 2; ++nt) {
        uint32_t vb[4];
        ldsm4t(vb, b_addr + (kt * 16 * VS + nt * 16) * 2);
        mma(acc[2 * nt], ah, vb[0], vb[1]);
        mma(acc[2 * nt + 1], ah, vb[2], vb[3]);
        mma(acc[2 * nt], al, vb[0], vb[1]);
        mma(acc[2 * nt + 1], al, vb[2], vb[3]);
      }
    }
  }
  float* S = a.add + (chunk_id(a.bt, b, blockIdx.x) * a.r.heads + h) * (size_t)D * V;
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int d = d0 + wd * 16 + g + 8 * r, v = wv * (VP / 2) + i * 8 + 2 * t;
      if (d < D && v < V) *reinterpret_cast<float2*>(S + (size_t)d * V + v) = make_float2(acc[i][2 * r], acc[i][2 * r + 1]);
    }
}

__global__ void __launch_bounds__(256) gla_scan_kernel(const Args a) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int D = a.r.dim, V = a.r.vdim, per_head = D * V, heads = a.r.heads, channels = heads * D;
  const int b = blockIdx.z, h = blockIdx.y, e = (blockIdx.x * 256 + threadIdx.x) * 4, t0 = a.bt.cu[b], n = a.bt.cu[b + 1] - t0;
  if (e >= per_head || n <= 0) return;
  const float* cum = a.cum + (size_t)t0 * channels + h * D + e / V;   // 4 values of one channel: V is a multiple of 8
  float* own = a.state + ((size_t)a.bt.slot[b] * heads + h) * per_head + e;
  float4 S = a.bt.pos0[b] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(own);
  const int chunks = (n + kChunk - 1) / kChunk;
  const float* p = a.add + (chunk_id(a.bt, b, 0) * heads + h) * (size_t)per_head + e;
  bf16* o = a.starts + (chunk_id(a.bt, b, 0) * heads + h) * (size_t)(2 * per_head) + e;
  const size_t step = (size_t)heads * per_head;
  auto total = [&](int c) { return cum[(size_t)(min((c + 1) * kChunk, n) - 1) * channels]; };
  float4 next = *reinterpret_cast<const float4*>(p);
  float ltot = total(0);
  for (int c = 0; c < chunks; ++c, p += step, o += 2 * step) {
    const float4 dl = next;
    const float f = expf(ltot);
    if (c + 1 < chunks) {
      next = *reinterpret_cast<const float4*>(p + step);
      ltot = total(c + 1);
    }
    const float hx = __bfloat162float(__float2bfloat16_rn(S.x)), hy = __bfloat162float(__float2bfloat16_rn(S.y));
    const float hz = __bfloat162float(__float2bfloat16_rn(S.z)), hw = __bfloat162float(__float2bfloat16_rn(S.w));
    *reinterpret_cast<uint2*>(o) = make_uint2(pack2(hx, hy), pack2(hz, hw));
    *reinterpret_cast<uint2*>(o + per_head) = make_uint2(pack2(S.x - hx, S.y - hy), pack2(S.z - hz, S.w - hw));
    S.x = f * S.x + dl.x; S.y = f * S.y + dl.y; S.z = f * S.z + dl.z; S.w = f * S.w + dl.w;
  }
  *reinterpret_cast<float4*>(own) = S;
}

template <int DP, int VP>
__global__ void __launch_bounds__(kThreads, 1) gla_output_kernel(const Args a) {
  constexpr int KS = DP + 8, VS = VP + 8, SR = 64, SLICES = DP / SR;   // SR: channels of the state per pass
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* ks = reinterpret_cast<bf16*>(smem_raw);      // [chunk][DP] keys, weighted to the end of their block
  bf16* buf = ks + kChunk * KS;                      // two tiles of 128 x VP, in turn: slices of the state ([high part, rest][SR][VP]), the values
  float* ends = reinterpret_cast<float*>(buf + 2 * kChunk * VS);   // [blocks][DP] b at the end of each block
  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.z, h = blockIdx.y, chunk = blockIdx.x, t0 = a.bt.cu[b], n = a.bt.cu[b + 1] - t0, first = chunk * kChunk;
  if (first >= n) return;
  const int len = min(kChunk, n - first), D = a.r.dim, V = a.r.vdim, channels = a.r.heads * D, V8 = V / 8;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const float kscale = 1.f / sqrtf((float)D);
  const float* cum = a.cum + (size_t)(t0 + first) * channels + h * D;
  const bf16* rows = a.proj + (size_t)(t0 + first) * a.stride;
  const bf16* S = a.starts + (chunk_id(a.bt, b, chunk) * a.r.heads + h) * (size_t)(2 * D * V);
  const bool has_state = chunk > 0 || a.bt.pos0[b] != 0;

  const int slices = has_state ? SLICES : 0;
  auto load = [&](int i) {   // tile i; columns past V and what lies outside the chunk become zeros
    bf16* dst = buf + (i & 1) * kChunk * VS;
    for (int e = tid; e < kChunk * (VP / 8); e += kThreads) {
      const int r = e / (VP / 8), c = e % (VP / 8);
      const bf16* src;
      bool ok = c < V8;
      if (i < slices) {
        const int d = i * SR + r % SR;
        ok = ok && d < D;
        src = S + ((size_t)(r / SR) * D + (ok ? d : 0)) * V + (ok ? c * 8 : 0);
      } else {
        ok = ok && r < len;
        src = rows + (size_t)(ok ? r : 0) * a.stride + a.v_off + (size_t)h * V + (ok ? c * 8 : 0);
      }
      cp16(smem_addr(dst + r * VS + c * 8), src, ok);
    }
    cp_commit();
  };
  load(0);
  if (slices > 0) load(1);
  for (int e = tid; e < kBlocks * DP; e += kThreads) {
    const int w = e / DP, d = e % DP;
    ends[e] = d < D ? cum[(size_t)min(w * kBlock + kBlock - 1, len - 1) * channels + d] : 0.f;
  }
  __syncthreads();
  {
    // a thread weighs two neighbouring channels of every RT-th token, 8 tokens' loads under way at once (from places that exist)
    constexpr int RT = kThreads / (DP / 2);
    const int d = tid % (DP / 2) * 2, dd = d < D ? d : 0;
    const float* cb = cum + dd;
    const bf16* kb = rows + a.k_off + (size_t)h * D + dd;
    for (int j0 = tid / (DP / 2); j0 < kChunk; j0 += 8 * RT) {
      float2 bj[8];
      uint32_t kv[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int j = min(j0 + i * RT, len - 1);
        bj[i] = *reinterpret_cast<const float2*>(cb + (size_t)j * channels);
        kv[i] = *reinterpret_cast<const uint32_t*>(kb + (size_t)j * a.stride);
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int j = j0 + i * RT;
        const float* en = ends + (j / kBlock) * DP + d;
        const bool ok = j < len && d < D;
        const float x = __uint_as_float(kv[i] << 16) * kscale * exp_fast(en[0] - bj[i].x);
        const float y = __uint_as_float(kv[i] & 0xFFFF0000u) * kscale * exp_fast(en[1] - bj[i].y);
        *reinterpret_cast<uint32_t*>(ks + j * KS + d) = ok ? pack2(x, y) : 0u;
      }
    }
  }
  // this warp's queries: rows g and g + 8 of block `warp`, times exp(b_i - b at the end of the block before)
  const int i0 = warp * kBlock;
  const bool busy = i0 < len;
  const float* ref = warp > 0 ? ends + (warp - 1) * DP : nullptr;
  float q[DP / 16][8];   // [k-step][row g: 2t, 2t + 1; row g + 8; the same 8 channels on]
  {
    const float* cb[2];
    const bf16* qb[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = min(i0 + g + 8 * r, len - 1);
      cb[r] = cum + (size_t)row * channels;
      qb[r] = rows + (size_t)row * a.stride + a.q_off + (size_t)h * D;
    }
#pragma unroll
    for (int k0 = 0; k0 < DP / 16; k0 += 2) {
      float2 bi[2][4];
      uint32_t qv[2][4];
#pragma unroll
      for (int k = 0; k < 2; ++k)
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int d = (k0 + k) * 16 + 2 * t + 8 * (u >> 1), dd = d < D ? d : 0;
          bi[k][u] = *reinterpret_cast<const float2*>(cb[u & 1] + dd);
          qv[k][u] = *reinterpret_cast<const uint32_t*>(qb[u & 1] + dd);
        }
#pragma unroll
      for (int k = 0; k < 2; ++k)
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int d = (k0 + k) * 16 + 2 * t + 8 * (u >> 1);
          const bool ok = d < D && i0 + g + 8 * (u & 1) < len;
          q[k0 + k][2 * u] = ok ? __uint_as_float(qv[k][u] << 16) * exp_fast(bi[k][u].x - (ref ? ref[d] : 0.f)) : 0.f;
          q[k0 + k][2 * u + 1] = ok ? __uint_as_float(qv[k][u] & 0xFFFF0000u) * exp_fast(bi[k][u].y - (ref ? ref[d + 1] : 0.f)) : 0.f;
        }
    }
  }
  bool steep = false;
  if (busy)
    for (int d = lane; d < D; d += 32) steep |= (ref ? ref[d] : 0.f) - ends[warp * DP + d] > kMaxSpan;
  steep = __any_sync(0xFFFFFFFFu, steep);
  float O[VP / 8][4];
#pragma unroll
  for (int i = 0; i < VP / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) O[i][e] = 0.f;
  const uint32_t k_lane = smem_addr(ks) + (((lane & 7) + ((lane >> 4) << 3)) * KS + ((lane >> 3) & 1) * 8) * 2;
  const uint32_t v_lane = (((lane & 7) + (((lane >> 3) & 1) << 3)) * VS + (lane >> 4) * 8) * 2;
  auto product = [&](const uint32_t (&pa)[4], uint32_t base) {   // O += 16 x 16 operand times 16 rows of a tile
#pragma unroll
    for (int nt = 0; nt < VP / 16; ++nt) {
      uint32_t vb[4];
      ldsm4t(vb, base + nt * 32);
      mma(O[2 * nt], pa, vb[0], vb[1]);
      mma(O[2 * nt + 1], pa, vb[2], vb[3]);
    }
  };
  // queries against the state at the chunk's start
#pragma unroll
  for (int sl = 0; sl < SLICES; ++sl) {
    if (sl >= slices) break;
    cp_wait<1>();       // the next tile may still be under way
    __syncthreads();
    if (busy) {
#pragma unroll
      for (int k = 0; k < SR / 16; ++k) {
        const int kt = sl * (SR / 16) + k;
        float f[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) f[u] = ref ? exp_fast(ref[kt * 16 + 2 * t + 8 * (u >> 1) + (u & 1)]) : 1.f;
        const uint32_t qa[4] = {pack2(q[kt][0] * f[0], q[kt][1] * f[1]), pack2(q[kt][2] * f[0], q[kt][3] * f[1]),
                                pack2(q[kt][4] * f[2], q[kt][5] * f[3]), pack2(q[kt][6] * f[2], q[kt][7] * f[3])};
        const uint32_t base = smem_addr(buf + (sl & 1) * kChunk * VS + k * 16 * VS) + v_lane;
        product(qa, base);
        product(qa, base + SR * VS * 2);
      }
    }
    __syncthreads();
    if (sl + 2 <= slices) load(sl + 2);
  }
  cp_wait<0>();
  __syncthreads();   // the values (and the keys) are in place
  if (!busy) return;
  // scores inside the chunk, block by block, and their product with the values
  const uint32_t values = smem_addr(buf + (slices & 1) * kChunk * VS) + v_lane;
#pragma unroll 1
  for (int J = 0; J <= warp; ++J) {
    float s[2][4] = {};
    if (J == warp && steep) {
      const bf16 *qg = rows + a.q_off + (size_t)h * D, *kg = rows + a.k_off + (size_t)h * D;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = i0 + g + 8 * (e >> 1), j = i0 + nt * 8 + 2 * t + (e & 1);
          float sum = 0.f;
          if (i < len && j <= i) {
#pragma unroll 1
            for (int d = 0; d < D; ++d)
              sum += to_f(qg[(size_t)i * a.stride + d]) * to_f(kg[(size_t)j * a.stride + d]) *
                     exp_fast(cum[(size_t)i * channels + d] - cum[(size_t)j * channels + d]);
          }
          s[nt][e] = sum * kscale;
        }
    } else {
#pragma unroll
      for (int kt = 0; kt < DP / 16; ++kt) {
        float f[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int d = kt * 16 + 2 * t + 8 * (u >> 1) + (u & 1);
          f[u] = exp_fast((ref ? ref[d] : 0.f) - ends[J * DP + d]);
        }
        const uint32_t qa[4] = {pack2(q[kt][0] * f[0], q[kt][1] * f[1]), pack2(q[kt][2] * f[0], q[kt][3] * f[1]),
                                pack2(q[kt][4] * f[2], q[kt][5] * f[3]), pack2(q[kt][6] * f[2], q[kt][7] * f[3])};
        uint32_t kf[4];
        ldsm4(kf, k_lane + (J * kBlock * KS + kt * 16) * 2);
        mma(s[0], qa, kf[0], kf[1]);
        mma(s[1], qa, kf[2], kf[3]);
      }
      if (J == warp) {
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (nt * 8 + 2 * t + (e & 1) > g + 8 * (e >> 1)) s[nt][e] = 0.f;
      }
    }
    const uint32_t pa[4] = {pack2(s[0][0], s[0][1]), pack2(s[0][2], s[0][3]), pack2(s[1][0], s[1][1]), pack2(s[1][2], s[1][3])};
    product(pa, values + J * kBlock * VS * 2);
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < VP / 8; ++i) sum += O[i][2 * r] * O[i][2 * r] + O[i][2 * r + 1] * O[i][2 * r + 1];
    const float f = a.r.out_scale / sqrtf(quad_sum(sum) / (float)V + a.r.eps);
    const int row = i0 + g + 8 * r;
    if (row >= len) continue;
    bf16* dst = a.act + (size_t)(t0 + first + row) * a.act_stride + (size_t)h * V;
    const bf16* gp = rows + (size_t)row * a.stride + a.g_off + (size_t)h * V;
    constexpr int U = VP / 8 < 16 ? VP / 8 : 16;   // loads under way at once (from places that exist)
#pragma unroll
    for (int i1 = 0; i1 < VP / 8; i1 += U) {
      uint32_t gw[U];
      float2 nw[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = (i1 + u) * 8 + 2 * t, cc = c < V ? c : 0;
        gw[u] = *reinterpret_cast<const uint32_t*>(gp + cc);
        nw[u] = a.r.norm ? *reinterpret_cast<const float2*>(a.r.norm + cc) : make_float2(1.f, 1.f);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = i1 + u, c = i * 8 + 2 * t;
        const float gx = __uint_as_float(gw[u] << 16), gy = __uint_as_float(gw[u] & 0xFFFF0000u);
        if (c < V)
          *reinterpret_cast<uint32_t*>(dst + c) = pack2(O[i][2 * r] * f * nw[u].x * (gx * sigmoid_fast(gx)), O[i][2 * r + 1] * f * nw[u].y * (gy * sigmoid_fast(gy)));
      }
    }
  }
}

template <typename K>
static int set_smem(K kernel, size_t smem) {
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return NQB200_ERR_LAUNCH;
  }
  return NQB200_OK;
}

template <int VP>
static int launch_chunk(const Args& a, int chunks, cudaStream_t st) {
  const size_t smem = (size_t)(2 * 64 * 72 + 64 * (VP + 8)) * sizeof(bf16);
  const int rc = set_smem(gla_chunk_kernel<VP>, smem);
  if (rc != NQB200_OK) return rc;
  return launch_overlapped(gla_chunk_kernel<VP>, dim3((unsigned)chunks, (unsigned)(a.r.heads * ((a.r.dim + 63) / 64)), (unsigned)a.bt.batch), dim3(kThreads), smem, st, a);
}
template <int DP, int VP>
static int launch_output(const Args& a, int chunks, cudaStream_t st) {
  const size_t smem = (size_t)(kChunk * (DP + 8) + 2 * kChunk * (VP + 8)) * sizeof(bf16) + (size_t)kBlocks * DP * sizeof(float);
  const int rc = set_smem(gla_output_kernel<DP, VP>, smem);
  if (rc != NQB200_OK) return rc;
  return launch_overlapped(gla_output_kernel<DP, VP>, dim3((unsigned)chunks, (unsigned)a.r.heads, (unsigned)a.bt.batch), dim3(kThreads), smem, st, a);
}

}  // namespace gla
}  // namespace nqb200

using namespace nqb200;

static int64_t gla_chunks(int64_t tokens, int64_t batch) { return tokens / gla::kChunk + batch; }

extern "C" int64_t nqb200_gla_scratch(const nqb200_retention_desc* r, int64_t tokens, int64_t batch) {
  if (!r) return 0;
  return tokens * r->heads * r->dim + 2 * gla_chunks(tokens, batch) * r->heads * r->dim * r->vdim;
}

extern "C" int nqb200_gla_prefill_supported(const nqb200_retention_desc* r, int64_t stride, int64_t off, int64_t act_stride, int64_t act_col) {
  return r && r->rank > 0 && r->rank <= 64 && r->rot <= 0 && r->heads > 0 && r->heads <= 16384 && r->dim > 0 && r->dim % 8 == 0 && r->dim <= 128 && r->vdim > 0 &&
                 r->vdim % 8 == 0 && r->vdim <= 256 && stride % 8 == 0 && off % 8 == 0 && act_stride % 2 == 0 && act_col % 2 == 0
             ? 1
             : 0;
}

extern "C" int nqb200_gla_prefill(const void* proj, int64_t stride, int64_t off, void* act, int64_t act_stride, int64_t act_col,
                                  const nqb200_retention_desc* r, float* state, float* scratch, const nqb200_batch* b, void* stream) {
  const int s = check_batch(b, false);
  if (s != NQB200_OK) return s;
  if (!nqb200_gla_prefill_supported(r, stride, off, act_stride, act_col) || !(r->tau > 0.f)) return NQB200_ERR_BAD_SHAPE;
  if (b->tokens == 0) return NQB200_OK;
  if (!proj || !act || !state || !scratch || !r->a2 || !r->a2_bias) return NQB200_ERR_NULL_POINTER;
  if (!aligned16(proj) || !aligned16(act) || !aligned16(state) || !aligned16(scratch)) return NQB200_ERR_MISALIGNED;
  cudaStream_t st = (cudaStream_t)stream;
  const int chunks = (b->max_len + gla::kChunk - 1) / gla::kChunk, channels = r->heads * r->dim;
  if (chunks > 65535) return NQB200_ERR_TOO_LARGE;
  gla::Args a = {};
  a.proj = (const bf16*)proj; a.stride = stride;
  a.q_off = (int)off; a.k_off = a.q_off + channels; a.v_off = a.k_off + channels; a.g_off = a.v_off + r->heads * r->vdim; a.l_off = a.g_off + r->heads * r->vdim;
  a.act = (bf16*)act + act_col; a.act_stride = act_stride; a.r = *r; a.state = state; a.bt = *b;
  a.cum = scratch;
  a.add = a.cum + (int64_t)b->tokens * channels;
  a.starts = reinterpret_cast<bf16*>(a.add + gla_chunks(b->tokens, b->batch) * channels * r->vdim);
  int rc = launch_overlapped(gla::gla_decay_kernel, dim3((unsigned)((channels + gla::kDecayChannels - 1) / gla::kDecayChannels), (unsigned)chunks, (unsigned)b->batch),
                             dim3(gla::kDecayChannels), (size_t)gla::kChunk * r->rank * sizeof(float), st, a);
  if (rc == NQB200_OK) rc = r->vdim <= 64 ? gla::launch_chunk<64>(a, chunks, st) : r->vdim <= 128 ? gla::launch_chunk<128>(a, chunks, st) : gla::launch_chunk<256>(a, chunks, st);
  if (rc == NQB200_OK)
    rc = launch_overlapped(gla::gla_scan_kernel, dim3((unsigned)((r->dim * r->vdim / 4 + 255) / 256), (unsigned)r->heads, (unsigned)b->batch), dim3(256), 0, st, a);
  if (rc != NQB200_OK) return rc;
#define NQB200_GLA(D)                                           \
  do {                                                          \
    if (r->vdim <= 64) return gla::launch_output<D, 64>(a, chunks, st);   \
    if (r->vdim <= 128) return gla::launch_output<D, 128>(a, chunks, st); \
    return gla::launch_output<D, 256>(a, chunks, st);           \
  } while (0)
  if (r->dim <= 64) NQB200_GLA(64);
  NQB200_GLA(128);
#undef NQB200_GLA
}
