// One decode step (one token per sequence) of the mixers that stand side by side in a layer, in one launch: chunked
// attention with its rotary embedding and K/V store, and retention with its norm and gate.
//
// Work is dealt to thread-block clusters: a cluster takes one (sequence, key/value head, group of query heads) of the
// attention and splits the visible keys over its CTAs, or one (sequence, head) of the retention and splits the value
// columns.  The CTAs of a cluster combine through distributed shared memory.
#include <cooperative_groups.h>
#include "mixers.cuh"

namespace cg = cooperative_groups;

namespace nqb200 {

constexpr int kDecThreads = 128;
constexpr int kDecTile = 128;      // keys per pass of a CTA
constexpr int kDecHeads = 8;       // query heads per cluster at most (columns of one mma)
constexpr int kDecMaxDim = 256;

struct DecodeArgs {
  const bf16* proj; int64_t stride;
  bf16* act; int64_t act_stride;
  nqb200_batch bt;
  // attention; att_clusters = kv_heads * head_groups per sequence (0: none)
  nqb200_attention at;
  const float* inv_freq; int rot;
  int q_off, k_off, v_off, a_col, att_clusters, head_groups;
  bf16* k_cache; bf16* v_cache;
  // retention (ret_heads 0: none)
  int ret_heads, rdim, rvdim, rq_off, rk_off, rv_off, rg_off, r_col;
  const float* decay; float* rstate;
  float eps, r_scale;
};

struct AttSmem {
  alignas(16) bf16 q[kDecHeads][kDecMaxDim + 8];
  alignas(16) bf16 knew[kDecMaxDim];
  float p[kDecHeads][kDecTile + 4];
  float cs[kDecMaxDim];
  float m[kDecHeads], l[kDecHeads], corr[kDecHeads];
  int rows[kDecTile];
  float out[kDecHeads][kDecMaxDim];           // this CTA's share, read by the cluster
  float red[kDecThreads * kDecHeads * 8];     // partial sums of the key groups
};

struct RetSmem {
  float q[1024], k[1024];
  float red[kDecThreads * 4];
  float o[1024];
  float ss, wsum[4];
};

__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// R: query heads of this cluster (compile-time bound RM).
template <int RM>
__device__ void attention_decode(const DecodeArgs& a, AttSmem& sm, int b, int unit, cg::cluster_group& cl) {
  const nqb200_attention& at = a.at;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rank = (int)cl.block_rank(), csize = (int)cl.num_blocks();
  const int per_kv = at.heads / at.kv_heads, kvh = unit / a.head_groups, hg = unit % a.head_groups;
  const int h0 = kvh * per_kv + hg * RM, R = min(RM, per_kv - hg * RM);   // query heads h0 .. h0 + R - 1
  const int D = at.dim, V = at.vdim, pos = a.bt.pos0[b];
  const int lo = at.chunk > 0 ? pos / at.chunk * at.chunk : 0, nk = pos - lo + 1;
  const int per = (nk + csize - 1) / csize, k0 = lo + rank * per, k1 = min(lo + nk, k0 + per);   // this CTA's keys
  const bf16* row = a.proj + (size_t)b * a.stride;
  const int half = a.rot / 2, dpad = (D + 31) / 32 * 32;

  for (int f = tid; f < half; f += kDecThreads) sincosf((float)pos * a.inv_freq[f], &sm.cs[half + f], &sm.cs[f]);
  for (int e = tid; e < kDecHeads * dpad; e += kDecThreads) sm.q[e / dpad][e % dpad] = __float2bfloat16_rn(0.f);
  if (tid < kDecHeads) { sm.m[tid] = -INFINITY; sm.l[tid] = 0.f; }
  __syncthreads();
  // rotate q (R heads) and, in the CTA that holds the newest key, k; that CTA also stores k and v
  const bool newest = k0 <= pos && pos < k1;
  const size_t nrow = newest ? kv_row(a.bt, b, pos) : 0;
  bf16* kdst = a.k_cache + (nrow * at.kv_heads + kvh) * D;
  bf16* vdst = a.v_cache + (nrow * at.kv_heads + kvh) * V;
  const int pairs = half + (D - a.rot), nvec = R + (newest ? 1 : 0);
  for (int e = tid; e < nvec * pairs; e += kDecThreads) {
    const int r = e / pairs, j = e % pairs;
    const bf16* src = r < R ? row + a.q_off + (size_t)(h0 + r) * D : row + a.k_off + (size_t)kvh * D;
    bf16* dst = r < R ? sm.q[r] : sm.knew;
    if (j < half) {
      const float u = to_f(src[j]), v = to_f(src[j + half]), c = sm.cs[j], s = sm.cs[half + j];
      dst[j] = __float2bfloat16_rn(u * c - v * s);
      dst[j + half] = __float2bfloat16_rn(v * c + u * s);
    } else {
      dst[j + half] = src[j + half];
    }
  }
  __syncthreads();
  if (newest && hg == 0) {   // every head group of the key/value head would write the same
    for (int d = tid; d < D; d += kDecThreads) kdst[d] = sm.knew[d];
    for (int d = tid; d < V; d += kDecThreads) vdst[d] = row[a.v_off + (size_t)kvh * V + d];
  }

  const int CG = V / 8, KG = kDecThreads / CG, cgi = tid % CG, kgi = tid / CG;   // 8 value columns x a key group per thread
  const bool pv = kgi < KG;
  float acc[RM][8];
#pragma unroll
  for (int r = 0; r < RM; ++r)
#pragma unroll
    for (int c = 0; c < 8; ++c) acc[r][c] = 0.f;
  const int g = lane >> 2, t = lane & 3;
  for (int j0 = k0; j0 < k1; j0 += kDecTile) {
    const int cnt = min(kDecTile, k1 - j0);
    __syncthreads();
    if (tid < cnt) sm.rows[tid] = (int)kv_row(a.bt, b, j0 + tid);
    __syncthreads();
    // scores: 16 keys per warp and turn, keys as rows of the mma, query heads as its columns
    for (int kk = warp * 16; kk < cnt; kk += 64) {
      const bf16* kp[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int key = kk + g + 8 * i;
        kp[i] = (key < cnt && j0 + key != pos) ? a.k_cache + ((size_t)sm.rows[key] * at.kv_heads + kvh) * D : sm.knew;
        if (key >= cnt) kp[i] = nullptr;
      }
      float c[4] = {0.f, 0.f, 0.f, 0.f};
      for (int d0 = 0; d0 < dpad; d0 += 32) {
        const int d = d0 + t * 8;
        uint4 ka = make_uint4(0, 0, 0, 0), kb = ka;
        if (d < D && kp[0]) ka = *reinterpret_cast<const uint4*>(kp[0] + d);
        if (d < D && kp[1]) kb = *reinterpret_cast<const uint4*>(kp[1] + d);
        const uint4 qv = *reinterpret_cast<const uint4*>(&sm.q[g][d]);
        mma_bf16(c, ka.x, kb.x, ka.y, kb.y, qv.x, qv.y);
        mma_bf16(c, ka.z, kb.z, ka.w, kb.w, qv.z, qv.w);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = kk + g + 8 * (e >> 1), r = t * 2 + (e & 1);
        float s = c[e] * at.scale;
        if (at.softcap > 0.f) s = at.softcap * tanhf(s / at.softcap);
        sm.p[r][key] = key < cnt ? s : -INFINITY;
      }
    }
    __syncthreads();
    // softmax of the tile: a warp per head
    for (int r = warp; r < R; r += 4) {
      float mx = -INFINITY;
      for (int i = lane; i < cnt; i += 32) mx = fmaxf(mx, sm.p[r][i]);
      const float m_old = sm.m[r], m_new = fmaxf(m_old, warp_max(mx));
      float s = 0.f;
      for (int i = lane; i < cnt; i += 32) {
        const float e = expf(sm.p[r][i] - m_new);
        sm.p[r][i] = e;
        s += e;
      }
      s = warp_sum(s);
      __syncwarp();
      if (lane == 0) {
        const float corr = expf(m_old - m_new);
        sm.corr[r] = corr;
        sm.m[r] = m_new;
        sm.l[r] = sm.l[r] * corr + s;
      }
    }
    __syncthreads();
    if (pv) {
#pragma unroll
      for (int r = 0; r < RM; ++r) {
        const float corr = r < R ? sm.corr[r] : 0.f;
#pragma unroll
        for (int c = 0; c < 8; ++c) acc[r][c] *= corr;
      }
#pragma unroll 4
      for (int i = kgi; i < cnt; i += KG) {
        const bf16* vp = (j0 + i != pos) ? a.v_cache + ((size_t)sm.rows[i] * at.kv_heads + kvh) * V : row + a.v_off + (size_t)kvh * V;
        float vf[8];
        if (j0 + i != pos) {
          const uint4 v = *reinterpret_cast<const uint4*>(vp + cgi * 8);
          const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
          for (int c = 0; c < 4; ++c) { vf[2 * c] = __uint_as_float(w[c] << 16); vf[2 * c + 1] = __uint_as_float(w[c] & 0xFFFF0000u); }
        } else {   // the new token's v stands in the projection, at any alignment
#pragma unroll
          for (int c = 0; c < 8; ++c) vf[c] = to_f(vp[cgi * 8 + c]);
        }
#pragma unroll
        for (int r = 0; r < RM; ++r) {
          if (r >= R) break;
          const float w = sm.p[r][i];
#pragma unroll
          for (int c = 0; c < 8; ++c) acc[r][c] += w * vf[c];
        }
      }
    }
  }
  __syncthreads();
  // sum over the key groups, then over the cluster's CTAs
  if (pv) {
#pragma unroll
    for (int r = 0; r < RM; ++r)
#pragma unroll
      for (int c = 0; c < 8; ++c)
        if (r < R) sm.red[(kgi * RM + r) * V + cgi * 8 + c] = acc[r][c];
  }
  __syncthreads();
  for (int e = tid; e < R * V; e += kDecThreads) {
    const int r = e / V, c = e % V;
    float s = 0.f;
    for (int k = 0; k < KG; ++k) s += sm.red[(k * RM + r) * V + c];
    sm.out[r][c] = s;
  }
  cl.sync();
  for (int e = rank * kDecThreads + tid; e < R * V; e += csize * kDecThreads) {
    const int r = e / V, c = e % V;
    const float sink = at.sink ? at.sink[h0 + r] : -INFINITY;
    float m = sink;
    for (int k = 0; k < csize; ++k) m = fmaxf(m, cl.map_shared_rank(&sm, k)->m[r]);
    float l = at.sink ? expf(sink - m) : 0.f, o = 0.f;
    for (int k = 0; k < csize; ++k) {
      const AttSmem* s = cl.map_shared_rank(&sm, k);
      const float f = expf(s->m[r] - m);      // 0 for a CTA without keys
      l += s->l[r] * f;
      o += s->out[r][c] * f;
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
  const float kscale = 1.f / sqrtf((float)D), d = a.decay[h];
  const bool fresh = a.bt.pos0[b] == 0;
  for (int e = tid; e < D; e += kDecThreads) {
    sm.q[e] = to_f(row[a.rq_off + (size_t)h * D + e]);
    sm.k[e] = to_f(row[a.rk_off + (size_t)h * D + e]) * kscale;
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
#pragma unroll 4
      for (int r = rgi; r < D; r += RG) {
        float* sp = st + (size_t)r * V + col;
        float s[VEC];
        if (VEC == 4) {
          float4 f = fresh ? make_float4(0, 0, 0, 0) : *reinterpret_cast<const float4*>(sp);
          s[0] = f.x; s[1 % VEC] = f.y; s[2 % VEC] = f.z; s[3 % VEC] = f.w;
        } else {
          s[0] = fresh ? 0.f : *sp;
        }
        const float kr = sm.k[r], qr = sm.q[r];
#pragma unroll
        for (int i = 0; i < VEC; ++i) { s[i] = d * s[i] + kr * v[i]; acc[i] += s[i] * qr; }
        if (VEC == 4) *reinterpret_cast<float4*>(sp) = make_float4(s[0], s[1 % VEC], s[2 % VEC], s[3 % VEC]);
        else *sp = s[0];
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
  if (tid == 0) sm.ss = sm.wsum[0] + sm.wsum[1] + sm.wsum[2] + sm.wsum[3];
  cl.sync();
  float tot = 0.f;
  for (int k = 0; k < csize; ++k) tot += cl.map_shared_rank(&sm, k)->ss;
  const float inv = a.r_scale / sqrtf(tot / (float)V + a.eps);
  for (int e = tid; e < ncol * VEC; e += kDecThreads) {
    const int c = c0 * VEC + e;
    const float gt = to_f(row[a.rg_off + (size_t)h * V + c]);
    a.act[(size_t)b * a.act_stride + a.r_col + (size_t)h * V + c] = __float2bfloat16_rn(sm.o[e] * inv * (gt * sigmoid_f(gt)));
  }
  cl.sync();
}

template <int RM, int VEC>
__global__ void __launch_bounds__(kDecThreads) mixer_decode_kernel(const DecodeArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  grid_launch_dependents();
  grid_dependency_wait();
  cg::cluster_group cl = cg::this_cluster();
  const int unit = blockIdx.y, b = blockIdx.z;
  if (unit < a.att_clusters) attention_decode<RM>(a, *reinterpret_cast<AttSmem*>(smem), b, unit, cl);
  else retention_decode<VEC>(a, *reinterpret_cast<RetSmem*>(smem), b, unit - a.att_clusters, cl);
}

template <int RM, int VEC>
static int launch_decode(const DecodeArgs& a, int csize, cudaStream_t st) {
  const size_t smem = sizeof(AttSmem) > sizeof(RetSmem) ? sizeof(AttSmem) : sizeof(RetSmem);
  if (cudaFuncSetAttribute(mixer_decode_kernel<RM, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
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
  if (cudaLaunchKernelEx(&cfg, mixer_decode_kernel<RM, VEC>, a) != cudaSuccess) {
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
  if (r && (r->heads <= 0 || r->dim <= 0 || r->dim > 1024 || r->vdim <= 0 || r->vdim > 1024)) return 0;
  return a || r ? 1 : 0;
}

extern "C" int nqb200_mixer_decode(const void* proj, int64_t stride, void* act, int64_t act_stride, const nqb200_attention* a,
                                   const float* inv_freq, int64_t rot, int64_t a_off, int64_t a_col, void* k_cache, void* v_cache,
                                   const nqb200_retention_desc* r, int64_t r_off, int64_t r_col, float* state, const nqb200_batch* b,
                                   void* stream) {
  int s = a ? check_batch(b, true) : NQB200_OK;
  if (s == NQB200_OK) s = r ? check_batch(b, false) : NQB200_OK;
  if (s != NQB200_OK) return s;
  if (!b) return NQB200_ERR_NULL_POINTER;
  if (!nqb200_mixer_decode_supported(a, r) || b->max_len > 1 || b->tokens != b->batch) return NQB200_ERR_BAD_SHAPE;
  if (b->tokens == 0) return NQB200_OK;
  if (!proj || !act || (a && (!k_cache || !v_cache || (rot > 0 && !inv_freq))) || (r && (!state || !r->decay))) return NQB200_ERR_NULL_POINTER;
  if (a && (rot < 0 || rot % 2 != 0 || rot > a->dim)) return NQB200_ERR_BAD_SHAPE;
  if (a && (!aligned16(k_cache) || !aligned16(v_cache))) return NQB200_ERR_MISALIGNED;
  if (r && !aligned16(state)) return NQB200_ERR_MISALIGNED;
  DecodeArgs p = {};
  p.proj = (const bf16*)proj; p.stride = stride; p.act = (bf16*)act; p.act_stride = act_stride; p.bt = *b;
  int csize = 1, rm = 1;
  int64_t units = 0;
  if (a) {
    const int per_kv = a->heads / a->kv_heads;
    rm = per_kv >= 5 ? 8 : per_kv >= 3 ? 4 : per_kv;
    p.at = *a;
    p.inv_freq = inv_freq; p.rot = (int)rot;
    p.q_off = (int)a_off; p.k_off = (int)(a_off + (int64_t)a->heads * a->dim); p.v_off = p.k_off + a->kv_heads * a->dim;
    p.a_col = (int)a_col; p.k_cache = (bf16*)k_cache; p.v_cache = (bf16*)v_cache;
    p.head_groups = (per_kv + rm - 1) / rm;
    p.att_clusters = a->kv_heads * p.head_groups;
    units += p.att_clusters;
    int64_t keys = (int64_t)b->table_width * b->block_size;
    if (a->chunk > 0 && a->chunk < keys) keys = a->chunk;
    while (csize < 8 && keys > (int64_t)csize * kDecTile) csize *= 2;
  }
  if (r) {
    p.ret_heads = r->heads; p.rdim = r->dim; p.rvdim = r->vdim;
    p.rq_off = (int)r_off; p.rk_off = p.rq_off + r->heads * r->dim; p.rv_off = p.rk_off + r->heads * r->dim;
    p.rg_off = p.rv_off + r->heads * r->vdim; p.r_col = (int)r_col;
    p.decay = r->decay; p.rstate = state; p.eps = r->eps; p.r_scale = r->out_scale;
    units += r->heads;
    int64_t bytes = (int64_t)r->dim * r->vdim * 4;    // a CTA moves about 16 KB of state each way
    while (csize < 8 && bytes > (int64_t)csize * 16384 && csize * 8 <= r->vdim) csize *= 2;
  }
  while (csize > 1 && units * b->batch * csize > kNumSMs * 8) csize /= 2;
  cudaStream_t st = (cudaStream_t)stream;
  const bool v4 = !r || r->vdim % 4 == 0;
#define NQB200_DEC(RM) return v4 ? launch_decode<RM, 4>(p, csize, st) : launch_decode<RM, 1>(p, csize, st)
  if (rm == 1) NQB200_DEC(1);
  if (rm == 2) NQB200_DEC(2);
  if (rm == 4) NQB200_DEC(4);
  NQB200_DEC(8);
#undef NQB200_DEC
}
