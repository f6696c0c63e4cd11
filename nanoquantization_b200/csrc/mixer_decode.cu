// One decode step (one token per sequence) of the mixers that stand side by side in a layer, in one launch: attention
// (softmax in chunks, or sigmoid weights) with its head norms, rotary embedding and K/V store, and retention or gated linear
// attention with its decays, norm and gate.
//
// Work is dealt to thread-block clusters: a cluster takes one (sequence, key/value head, group of query heads) of the
// attention and splits the visible keys over its CTAs, or one (sequence, head) of the retention and splits the value
// columns.  The CTAs of a cluster combine through distributed shared memory.
#include <cooperative_groups.h>
#include "mixers.cuh"

namespace cg = cooperative_groups;

namespace nqb200 {

constexpr int kDecThreads = 256;
constexpr int kDecMaxTile = 128;   // keys per pass of a CTA at most: 16 per warp
constexpr int kDecStages = 2;      // passes in the ring
constexpr int kDecHeads = 8;       // query heads per cluster at most (columns of one mma)
constexpr int kDecMaxDim = 256;
constexpr int kDecPS = kDecMaxTile + 8;

struct DecodeArgs {
  const bf16* proj; int64_t stride;
  bf16* act; int64_t act_stride;
  nqb200_batch bt;
  // attention; att_clusters = kv_heads * head_groups per sequence (0: none)
  nqb200_attention at;
  nqb200_rope rope;
  int q_off, k_off, v_off, a_col, att_clusters, head_groups;
  bf16* k_cache; bf16* v_cache;
  // retention (ret_heads 0: none)
  int ret_heads, rdim, rvdim, rq_off, rk_off, rv_off, rg_off, rl_off, r_col;
  nqb200_retention_desc rd;
  float* rstate;
};

// Fixed part of the attention's shared memory; the key / value ring follows it.
struct AttSmem {
  alignas(16) bf16 q[kDecHeads][kDecMaxDim + 8];
  alignas(16) bf16 p[16][kDecPS];             // weights, rows 8 .. 15 stay zero
  alignas(16) bf16 knew[kDecMaxDim];
  float s[kDecHeads][kDecMaxTile + 4];
  float cs[kDecMaxDim];
  int rows[4][kDecMaxTile];                   // cache rows of the keys of four successive tiles
  float m[kDecHeads], l[kDecHeads], corr[kDecHeads];
  float out[kDecHeads][kDecMaxDim];           // this CTA's share, read by the cluster
  float inv[kDecHeads + 1];                   // 1 / rms of the query heads and the new key
};

constexpr int kDecMaxRank = 512;
struct RetSmem {
  float q[1024], k[1024], d[1024];
  float low[kDecMaxRank];
  float red[kDecThreads * 4];
  float o[1024];
  float ss, wsum[kDecThreads / 32];
};

__device__ __forceinline__ uint32_t dec_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void dec_cp16(uint32_t dst, const void* src, bool ok) {
  const int n = ok ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n));
}
__device__ __forceinline__ void dec_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void dec_ldsm4(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void dec_ldsm4t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void dec_ldsm2(uint32_t (&r)[2], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(a));
}

__host__ __device__ constexpr int att_ks(int dim) { return (dim + 15) / 16 * 16 + 8; }   // row strides of the ring, in elements
__host__ __device__ constexpr int att_stage(int dim, int vp, int tile) { return tile * (att_ks(dim) + vp + 8); }

// VP: value columns padded to 64, 128 or 256; a warp owns a quarter of them and half of a tile's keys.
template <int VP, int TILE>
__device__ void attention_decode(const DecodeArgs& a, uint8_t* smem, int b, int unit, cg::cluster_group& cl) {
  AttSmem& sm = *reinterpret_cast<AttSmem*>(smem);
  bf16* ring = reinterpret_cast<bf16*>(smem + sizeof(AttSmem));
  const nqb200_attention& at = a.at;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rank = (int)cl.block_rank(), csize = (int)cl.num_blocks();
  const int per_kv = at.heads / at.kv_heads, kvh = unit / a.head_groups, hg = unit % a.head_groups;
  const int h0 = kvh * per_kv + hg * kDecHeads, R = min(kDecHeads, per_kv - hg * kDecHeads);   // query heads h0 .. h0 + R - 1
  const int D = at.dim, V = at.vdim, pos = a.bt.pos0[b];
  const int lo = at.chunk > 0 ? pos / at.chunk * at.chunk : 0, nk = pos - lo + 1;
  const int per = (nk + csize - 1) / csize, k0 = lo + rank * per, k1 = min(lo + nk, k0 + per);   // this CTA's keys
  const int tiles = k1 > k0 ? (k1 - k0 + TILE - 1) / TILE : 0;
  const int KS = att_ks(D), D8 = D / 8, V8 = V / 8, half = a.rope.rot / 2;
  constexpr int VS = VP + 8, NT = VP / 32;       // n-tiles of 8 columns per warp
  const bf16* row = a.proj + (size_t)b * a.stride;
  const bool newest = k0 <= pos && pos < k1;

  auto load_tile = [&](int i) {
    if (i < tiles) {
      bf16* kd = ring + (size_t)(i % kDecStages) * att_stage(D, VP, TILE);
      bf16* vd = kd + TILE * KS;
      // neighbouring threads copy neighbouring 16-byte pieces of a row
      const int j0 = k0 + i * TILE;
      auto copy = [&](bf16* dst, int dstride, const bf16* cache, int n8, int size) {
        const int dk = kDecThreads / n8, dc = kDecThreads % n8;
        for (int key = tid / n8, c = tid % n8; key < TILE;) {
          dec_cp16(dec_smem(dst + key * dstride + c * 8), cache + ((size_t)sm.rows[i & 3][key] * at.kv_heads + kvh) * size + c * 8,
                   j0 + key < k1 && j0 + key != pos);
          key += dk;
          c += dc;
          if (c >= n8) { c -= n8; ++key; }
        }
      };
      copy(kd, KS, a.k_cache, D8, D);
      copy(vd, VS, a.v_cache, V8, V);
    }
    asm volatile("cp.async.commit_group;");
  };
  auto find_rows = [&](int first, int count) {   // of tiles first .. first + count - 1
    for (int e = tid; e < count * TILE; e += kDecThreads) {
      const int i = first + e / TILE, key = e % TILE;
      if (i < tiles) sm.rows[i & 3][key] = (int)kv_row(a.bt, b, min(k0 + i * TILE + key, k1 - 1));
    }
  };
  find_rows(0, 4);
  __syncthreads();
#pragma unroll
  for (int i = 0; i < kDecStages - 1; ++i) load_tile(i);

  // while those are under way: padding columns, the rotated queries and (in the CTA that holds the newest key) key
  for (int e = tid; e < kDecStages * TILE * (KS - 8 - D); e += kDecThreads) {
    const int r = e / (KS - 8 - D), c = e % (KS - 8 - D);
    ring[(size_t)(r / TILE) * att_stage(D, VP, TILE) + (r % TILE) * KS + D + c] = __float2bfloat16_rn(0.f);
  }
  for (int e = tid; e < kDecStages * TILE * (VP - V); e += kDecThreads) {
    const int r = e / (VP - V), c = e % (VP - V);
    ring[(size_t)(r / TILE) * att_stage(D, VP, TILE) + TILE * KS + (r % TILE) * VS + V + c] = __float2bfloat16_rn(0.f);
  }
  for (int e = tid; e < kDecHeads * (KS - 8); e += kDecThreads) sm.q[e / (KS - 8)][e % (KS - 8)] = __float2bfloat16_rn(0.f);
  for (int e = tid; e < 16 * kDecPS; e += kDecThreads) sm.p[e / kDecPS][e % kDecPS] = __float2bfloat16_rn(0.f);
  for (int f = tid; f < half; f += kDecThreads) sincosf((float)pos * a.rope.inv_freq[f], &sm.cs[half + f], &sm.cs[f]);
  if (tid < kDecHeads) { sm.m[tid] = -INFINITY; sm.l[tid] = 0.f; }
  const int pairs = half + (D - a.rope.rot), nvec = R + (newest ? 1 : 0);
  auto vec = [&](int r) { return r < R ? row + a.q_off + (size_t)(h0 + r) * D : row + a.k_off + (size_t)kvh * D; };
  if (a.rope.q_norm) {
    for (int r = warp; r < nvec; r += kDecThreads / 32) {
      const bf16* src = vec(r);
      float ss = 0.f;
      for (int d = lane; d < D; d += 32) { const float x = to_f(src[d]); ss += x * x; }
      ss = warp_sum(ss);
      if (lane == 0) sm.inv[r] = 1.f / sqrtf(ss / (float)D + a.rope.eps);
    }
  }
  __syncthreads();
  for (int e = tid; e < nvec * pairs; e += kDecThreads) {
    const int r = e / pairs, j = e % pairs;
    const bf16* src = vec(r);
    bf16* dst = r < R ? sm.q[r] : sm.knew;
    const float* w = r < R ? a.rope.q_norm : a.rope.k_norm;
    const float inv = w ? sm.inv[r] : 1.f;
    if (j < half) {
      const int x = a.rope.interleaved ? 2 * j : j, y = a.rope.interleaved ? x + 1 : j + half;
      float u = to_f(src[x]), v = to_f(src[y]);
      const float c = sm.cs[j], s = sm.cs[half + j];
      if (w) { u = u * inv * w[x]; v = v * inv * w[y]; }
      dst[x] = __float2bfloat16_rn(u * c - v * s);
      dst[y] = __float2bfloat16_rn(v * c + u * s);
    } else {
      dst[j + half] = w ? __float2bfloat16_rn(to_f(src[j + half]) * inv * w[j + half]) : src[j + half];
    }
  }
  float factor[2], shift[2];   // of this lane's two query heads in the score product
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int r = (lane & 3) * 2 + u;
    factor[u] = at.scale * (at.temp && r < R ? at.temp[h0 + r] : 1.f);
    shift[u] = at.bias && r < R ? at.bias[h0 + r] : 0.f;
  }
  const float inv_cap = at.softcap > 0.f ? 1.f / at.softcap : 0.f;
  const uint32_t k_lane = (uint32_t)((warp * 16 + (lane & 15)) * KS + (lane >> 4) * 8) * 2;
  const int quarter = warp & 3, half_keys = (warp >> 2) * (TILE / 2);
  const uint32_t v_lane = (uint32_t)((half_keys + (lane & 7) + (((lane >> 3) & 1) << 3)) * VS + quarter * (VP / 4) + (lane >> 4) * 8) * 2;
  const uint32_t q_addr = dec_smem(&sm.q[lane & 7][((lane >> 3) & 1) * 8]);
  const uint32_t p_addr = dec_smem(&sm.p[lane & 15][half_keys + (lane >> 4) * 8]);
  const int g = lane >> 2, t = lane & 3;
  float O[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) O[i][e] = 0.f;

  for (int i = 0; i < tiles; ++i) {
    asm volatile("cp.async.wait_group %0;" ::"n"(kDecStages - 2));
    __syncthreads();               // tile i has landed for every thread; tile i - 1 is no longer read
    load_tile(i + kDecStages - 1);
    find_rows(i + 4, 1);           // over tile i's, whose loads are done; read after the next barrier at the earliest
    const int j0 = k0 + i * TILE, cnt = min(TILE, k1 - j0);
    bf16* kt = ring + (size_t)(i % kDecStages) * att_stage(D, VP, TILE);
    bf16* vt = kt + TILE * KS;
    if (pos >= j0 && pos < j0 + cnt) {   // the newest key and value: into the tile, and into the cache
      const size_t nrow = kv_row(a.bt, b, pos) * at.kv_heads + kvh;
      for (int d = tid; d < D; d += kDecThreads) {
        kt[(pos - j0) * KS + d] = sm.knew[d];
        if (hg == 0) a.k_cache[nrow * D + d] = sm.knew[d];
      }
      for (int d = tid; d < V; d += kDecThreads) {
        const bf16 v = row[a.v_off + (size_t)kvh * V + d];
        vt[(pos - j0) * VS + d] = v;
        if (hg == 0) a.v_cache[nrow * V + d] = v;
      }
      __syncthreads();
    }
    // scores: keys as rows of the mma, query heads as its columns; 16 keys per warp
    if (warp * 16 < TILE) {
      float c[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t ka = dec_smem(kt) + k_lane;
#pragma unroll 4
      for (int d = 0; d < KS - 8; d += 16) {
        uint32_t kf[4], qf[2];
        dec_ldsm4(kf, ka + d * 2);
        dec_ldsm2(qf, q_addr + d * 2);
        dec_mma(c, kf, qf[0], qf[1]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = warp * 16 + g + 8 * (e >> 1), r = t * 2 + (e & 1);
        float s = c[e] * factor[e & 1] + shift[e & 1];
        if (at.sigmoid) {
          sm.p[r][key] = __float2bfloat16_rn(key < cnt ? sigmoid_fast(s) : 0.f);
          continue;
        }
        if (at.softcap > 0.f) s = at.softcap * tanh_fast(s * inv_cap);
        sm.s[r][key] = key < cnt ? s : -INFINITY;
      }
    }
    __syncthreads();
    // softmax of the tile: a head per warp, TILE / 32 keys per lane
    if (warp < R && !at.sigmoid) {
      float x[TILE / 32], mx = -INFINITY, sum = 0.f;
#pragma unroll
      for (int k = 0; k < TILE / 32; ++k) { x[k] = sm.s[warp][lane + 32 * k]; mx = fmaxf(mx, x[k]); }
      const float m_old = sm.m[warp], m_new = fmaxf(m_old, warp_max(mx));
#pragma unroll
      for (int k = 0; k < TILE / 32; ++k) {
        x[k] = exp_fast(x[k] - m_new);
        sum += x[k];
        sm.p[warp][lane + 32 * k] = __float2bfloat16_rn(x[k]);
      }
      sum = warp_sum(sum);
      if (lane == 0) {
        const float corr = exp_fast(m_old - m_new);
        sm.corr[warp] = corr;
        sm.m[warp] = m_new;
        sm.l[warp] = sm.l[warp] * corr + sum;
      }
    }
    if (!at.sigmoid) {
      __syncthreads();
      const float corr = g < R ? sm.corr[g] : 0.f;
#pragma unroll
      for (int n = 0; n < NT; ++n) { O[n][0] *= corr; O[n][1] *= corr; }
    }
    const uint32_t va = dec_smem(vt) + v_lane;
#pragma unroll
    for (int kk = 0; kk < TILE / 32; ++kk) {
      uint32_t pf[4];
      dec_ldsm4(pf, p_addr + kk * 32);
#pragma unroll
      for (int n = 0; n < NT / 2; ++n) {
        uint32_t vf[4];
        dec_ldsm4t(vf, va + (kk * 16 * VS + n * 16) * 2);
        dec_mma(O[2 * n], pf, vf[0], vf[1]);
        dec_mma(O[2 * n + 1], pf, vf[2], vf[3]);
      }
    }
  }
  asm volatile("cp.async.wait_group 0;");
  // the two halves of the keys, one after the other
  for (int half_no = 0; half_no < 2; ++half_no) {
    if ((warp >> 2) == half_no) {
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        float2* o = reinterpret_cast<float2*>(&sm.out[g][quarter * (VP / 4) + n * 8 + 2 * t]);
        *o = half_no ? make_float2(o->x + O[n][0], o->y + O[n][1]) : make_float2(O[n][0], O[n][1]);
      }
    }
    __syncthreads();
  }
  cl.sync();
  for (int e = rank * kDecThreads + tid; e < R * V; e += csize * kDecThreads) {
    const int r = e / V, c = e % V;
    const float sink = at.sink ? at.sink[h0 + r] : -INFINITY;
    float pm[8], pl[8], po[8], m = sink;   // all of the cluster's shares at once
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const AttSmem* s = cl.map_shared_rank(&sm, k < csize ? k : 0);
      pm[k] = k < csize ? s->m[r] : -INFINITY;
      pl[k] = s->l[r];
      po[k] = s->out[r][c];
    }
    if (at.sigmoid) {
      float o = 0.f;
#pragma unroll
      for (int k = 0; k < 8; ++k) o += k < csize ? po[k] : 0.f;
      a.act[(size_t)b * a.act_stride + a.a_col + (size_t)(h0 + r) * V + c] = __float2bfloat16_rn(o * at.out_scale);
      continue;
    }
#pragma unroll
    for (int k = 0; k < 8; ++k) m = fmaxf(m, pm[k]);
    float l = at.sink ? expf(sink - m) : 0.f, o = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const float f = expf(pm[k] - m);      // 0 for a CTA without keys, and beyond the cluster
      l += pl[k] * f;
      o += po[k] * f;
    }
    a.act[(size_t)b * a.act_stride + a.a_col + (size_t)(h0 + r) * V + c] = __float2bfloat16_rn(o / l * at.out_scale);
  }
  cl.sync();   // peers may still read this CTA's shared memory
}

// VEC columns per thread (4 where the value size allows 16-byte rows).
template <int VEC>
__device__ void retention_decode(const DecodeArgs& a, RetSmem& sm, int b, int h, cg::cluster_group& cl) {
  const int tid = threadIdx.x, rank = (int)cl.block_rank(), csize = (int)cl.num_blocks();
  const int D = a.rdim, V = a.rvdim;
  const int quads = V / VEC, per = (quads + csize - 1) / csize;                 // column groups of one CTA
  const int c0 = min(rank * per, quads), ncol = min(per, quads - c0);
  const bf16* row = a.proj + (size_t)b * a.stride;
  const float kscale = 1.f / sqrtf((float)D);
  const int pos = a.bt.pos0[b], half = a.rd.rot / 2;
  const bool fresh = pos == 0;
  const bf16 *qr = row + a.rq_off + (size_t)h * D, *kr = row + a.rk_off + (size_t)h * D;
  for (int e = tid; e < half; e += kDecThreads) {
    float s, c;
    sincosf((float)pos * a.rd.inv_freq[e], &s, &c);
    const float qu = to_f(qr[e]), qv = to_f(qr[e + half]), ku = to_f(kr[e]), kv = to_f(kr[e + half]);
    sm.q[e] = qu * c - qv * s;
    sm.q[e + half] = qv * c + qu * s;
    sm.k[e] = (ku * c - kv * s) * kscale;
    sm.k[e + half] = (kv * c + ku * s) * kscale;
  }
  for (int e = 2 * half + tid; e < D; e += kDecThreads) {
    sm.q[e] = to_f(qr[e]);
    sm.k[e] = to_f(kr[e]) * kscale;
  }
  if (a.rd.rank > 0) {
    for (int e = tid; e < a.rd.rank; e += kDecThreads) sm.low[e] = to_f(row[a.rl_off + e]);
    __syncthreads();
    const bf16* a2 = reinterpret_cast<const bf16*>(a.rd.a2) + (size_t)h * D * a.rd.rank;
    for (int e = tid; e < D; e += kDecThreads) {
      float z = 0.f;
      for (int r = 0; r < a.rd.rank; ++r) z += sm.low[r] * to_f(a2[(size_t)e * a.rd.rank + r]);
      sm.d[e] = expf(log_sigmoid_f(z + a.rd.a2_bias[h * D + e]) / a.rd.tau);
    }
  } else {
    for (int e = tid; e < D; e += kDecThreads) sm.d[e] = a.rd.decay[h];
  }
  __syncthreads();
  float* st = a.rstate + ((size_t)a.bt.slot[b] * a.ret_heads + h) * D * V;
  float ss = 0.f;
  for (int cb = 0; cb < ncol; cb += kDecThreads) {   // one pass unless a CTA has more than 128 column groups
    const int width = min(ncol - cb, kDecThreads), RG = kDecThreads / width, cgi = tid % width, rgi = tid / width;
    const int col = (c0 + cb + cgi) * VEC;
    float acc[VEC], v[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) acc[i] = 0.f;
    if (rgi < RG) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = to_f(row[a.rv_off + (size_t)h * V + col + i]);
      constexpr int U = 16;   // rows under way per thread
      for (int r0 = rgi; r0 < D; r0 += U * RG) {
        float S[U][VEC];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int r = r0 + u * RG;
          const float* sp = st + (size_t)r * V + col;
          if (VEC == 4) {
            const float4 f = (fresh || r >= D) ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(sp);
            S[u][0] = f.x; S[u][1 % VEC] = f.y; S[u][2 % VEC] = f.z; S[u][3 % VEC] = f.w;
          } else {
            S[u][0] = (fresh || r >= D) ? 0.f : *sp;
          }
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int r = r0 + u * RG;
          if (r >= D) break;
          const float kr = sm.k[r], qr = sm.q[r], d = sm.d[r];
#pragma unroll
          for (int i = 0; i < VEC; ++i) { S[u][i] = d * S[u][i] + kr * v[i]; acc[i] += S[u][i] * qr; }
          float* sp = st + (size_t)r * V + col;
          if (VEC == 4) *reinterpret_cast<float4*>(sp) = make_float4(S[u][0], S[u][1 % VEC], S[u][2 % VEC], S[u][3 % VEC]);
          else *sp = S[u][0];
        }
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) sm.red[(rgi * width + cgi) * VEC + i] = acc[i];
    }
    __syncthreads();
    for (int e = tid; e < width * VEC; e += kDecThreads) {
      float o = 0.f;
      for (int r = 0; r < RG; ++r) o += sm.red[r * width * VEC + e];
      sm.o[cb * VEC + e] = o;
      ss += o * o;
    }
    __syncthreads();
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) sm.wsum[tid >> 5] = ss;
  __syncthreads();
  if (tid == 0) {
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < kDecThreads / 32; ++w) s += sm.wsum[w];
    sm.ss = s;
  }
  cl.sync();
  float tot = 0.f;
  for (int k = 0; k < csize; ++k) tot += cl.map_shared_rank(&sm, k)->ss;
  const float inv = a.rd.out_scale / sqrtf(tot / (float)V + a.rd.eps);
  for (int e = tid; e < ncol * VEC; e += kDecThreads) {
    const int c = c0 * VEC + e;
    const float gt = to_f(row[a.rg_off + (size_t)h * V + c]);
    a.act[(size_t)b * a.act_stride + a.r_col + (size_t)h * V + c] = __float2bfloat16_rn(sm.o[e] * inv * (a.rd.norm ? a.rd.norm[c] : 1.f) * (gt * sigmoid_f(gt)));
  }
  cl.sync();
}

template <int VP, int VEC, int TILE>
__global__ void __launch_bounds__(kDecThreads, 1) mixer_decode_kernel(const DecodeArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  grid_launch_dependents();
  grid_dependency_wait();
  cg::cluster_group cl = cg::this_cluster();
  const int unit = blockIdx.y, b = blockIdx.z;
  if (unit < a.att_clusters) attention_decode<VP, TILE>(a, smem, b, unit, cl);
  else retention_decode<VEC>(a, *reinterpret_cast<RetSmem*>(smem), b, unit - a.att_clusters, cl);
}

template <int VP, int VEC, int TILE>
static int launch_decode(const DecodeArgs& a, int csize, cudaStream_t st) {
  size_t smem = a.ret_heads > 0 ? sizeof(RetSmem) : 0;
  const size_t att = a.att_clusters > 0 ? sizeof(AttSmem) + (size_t)kDecStages * att_stage(a.at.dim, VP, TILE) * sizeof(bf16) : 0;
  if (att > smem) smem = att;
  if (cudaFuncSetAttribute(mixer_decode_kernel<VP, VEC, TILE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return NQB200_ERR_LAUNCH;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)csize, (unsigned)(a.att_clusters + a.ret_heads), (unsigned)a.bt.batch);
  cfg.blockDim = dim3(kDecThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = (unsigned)csize;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  if (cudaLaunchKernelEx(&cfg, mixer_decode_kernel<VP, VEC, TILE>, a) != cudaSuccess) {
    cudaGetLastError();
    return NQB200_ERR_LAUNCH;
  }
  return NQB200_OK;
}

}  // namespace nqb200

using namespace nqb200;

extern "C" int nqb200_mixer_decode_supported(const nqb200_attention* a, const nqb200_retention_desc* r) {
  if (a && (a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads != 0 || a->dim <= 0 || a->dim % 8 != 0 || a->dim > kDecMaxDim ||
            a->vdim <= 0 || a->vdim % 8 != 0 || a->vdim > kDecMaxDim))
    return 0;
  if (r && (r->heads <= 0 || r->dim <= 0 || r->dim > 1024 || r->vdim <= 0 || r->vdim > 1024 || r->rank > kDecMaxRank || r->rot < 0 || r->rot % 2 != 0 || r->rot > r->dim)) return 0;
  return a || r ? 1 : 0;
}

extern "C" int nqb200_mixer_decode(const void* proj, int64_t stride, void* act, int64_t act_stride, const nqb200_attention* a,
                                   const nqb200_rope* rope, int64_t a_off, int64_t v_off, int64_t a_col, void* k_cache, void* v_cache,
                                   const nqb200_retention_desc* r, int64_t r_off, int64_t r_col, float* state, const nqb200_batch* b,
                                   void* stream) {
  int s = a ? check_batch(b, true) : NQB200_OK;
  if (s == NQB200_OK) s = r ? check_batch(b, false) : NQB200_OK;
  if (s != NQB200_OK) return s;
  if (!b) return NQB200_ERR_NULL_POINTER;
  if (!nqb200_mixer_decode_supported(a, r) || b->max_len > 1 || b->tokens != b->batch) return NQB200_ERR_BAD_SHAPE;
  if (b->tokens == 0) return NQB200_OK;
  if (!proj || !act || (a && (!k_cache || !v_cache || !rope || (rope->rot > 0 && !rope->inv_freq) || (rope->q_norm && !rope->k_norm))) ||
      (r && (!state || (r->rot > 0 && !r->inv_freq) || (r->rank > 0 ? !r->a2 || !r->a2_bias : !r->decay))))
    return NQB200_ERR_NULL_POINTER;
  if (a && (rope->rot < 0 || rope->rot % 2 != 0 || rope->rot > a->dim || (a->sigmoid && (a->sink || a->softcap > 0.f)))) return NQB200_ERR_BAD_SHAPE;
  if (r && r->rank > 0 && !(r->tau > 0.f)) return NQB200_ERR_BAD_SHAPE;
  if (a && (!aligned16(k_cache) || !aligned16(v_cache))) return NQB200_ERR_MISALIGNED;
  if (r && !aligned16(state)) return NQB200_ERR_MISALIGNED;
  if (a && r && (int64_t)(a->kv_heads + r->heads) * b->batch > kNumSMs) {
    // more than one wave: each with the shared memory and the cluster size that suit it
    const int rc = nqb200_mixer_decode(proj, stride, act, act_stride, a, rope, a_off, v_off, a_col, k_cache, v_cache, nullptr, 0, 0, nullptr, b, stream);
    return rc != NQB200_OK ? rc
                           : nqb200_mixer_decode(proj, stride, act, act_stride, nullptr, nullptr, 0, 0, 0, nullptr, nullptr, r, r_off, r_col, state, b, stream);
  }
  DecodeArgs p = {};
  p.proj = (const bf16*)proj; p.stride = stride; p.act = (bf16*)act; p.act_stride = act_stride; p.bt = *b;
  int csize = 1, want = 1;
  int64_t units = 0;
  if (a) {
    const int per_kv = a->heads / a->kv_heads;
    p.at = *a;
    p.rope = *rope;
    p.q_off = (int)a_off; p.k_off = (int)(a_off + (int64_t)a->heads * a->dim); p.v_off = (int)v_off;
    p.a_col = (int)a_col; p.k_cache = (bf16*)k_cache; p.v_cache = (bf16*)v_cache;
    p.head_groups = (per_kv + kDecHeads - 1) / kDecHeads;
    p.att_clusters = a->kv_heads * p.head_groups;
    units += p.att_clusters;
    int64_t keys = (int64_t)b->table_width * b->block_size;
    if (a->chunk > 0 && a->chunk < keys) keys = a->chunk;
    while (want < 8 && keys > (int64_t)want * 64) want *= 2;
  }
  if (r) {
    p.ret_heads = r->heads; p.rdim = r->dim; p.rvdim = r->vdim;
    p.rq_off = (int)r_off; p.rk_off = p.rq_off + r->heads * r->dim; p.rv_off = p.rk_off + r->heads * r->dim;
    p.rg_off = p.rv_off + r->heads * r->vdim; p.rl_off = p.rg_off + r->heads * r->vdim; p.r_col = (int)r_col;
    p.rd = *r; p.rstate = state;
    units += r->heads;
    while (want < 8 && (int64_t)r->dim * r->vdim * 4 > (int64_t)want * 16384 && want * 8 <= r->vdim) want *= 2;
  }
  // about one CTA of attention per SM (its ring takes most of the shared memory), and no more than there is work for
  while (csize < want && units * b->batch * csize * 2 <= (a ? kNumSMs * 3 / 2 : kNumSMs * 4)) csize *= 2;
  cudaStream_t st = (cudaStream_t)stream;
  const bool v4 = !r || r->vdim % 4 == 0;
  // 128 keys a pass where two stages of them fit
#define NQB200_DEC(VP, TILE) return v4 ? launch_decode<VP, 4, TILE>(p, csize, st) : launch_decode<VP, 1, TILE>(p, csize, st)
  const bool big = a && a->dim + a->vdim > 256;
  if (!a || (a->vdim <= 64 && !big)) NQB200_DEC(64, 128);
  if (a->vdim <= 128 && !big) NQB200_DEC(128, 128);
  if (a->vdim <= 128) NQB200_DEC(128, 64);
  NQB200_DEC(256, 64);
#undef NQB200_DEC
}
