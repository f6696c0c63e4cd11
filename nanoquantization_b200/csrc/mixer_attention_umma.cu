// Chunk-masked attention of prompts on the 5th-generation tensor cores (head sizes 64 and 128, cache pages of a
// multiple of 128 tokens); what it computes is stated at nqb200_chunk_attention.
//
// One CTA takes 256 queries of one head as two tiles of 128 and walks over key tiles of 128.
//   warp 0        TMA: Q once, then a two-stage ring of K tiles and one of V tiles, straight from the pages.
//   warp 1        one thread issues tcgen05.mma: S = Q K^T (both operands in shared memory) and O += P V (P in
//                 tensor memory, V in shared memory as it lies there: the operand's rows are keys).
//   warps 4-7     softmax of tile 0, a thread per query row; warps 8-11 the same for tile 1.
// Tensor memory holds S of both tiles (128 columns each) and O of both; P overwrites the first half of its S.  The two
// tiles take turns on the tensor pipe while the other one's softmax runs.  The running maximum is only moved (and O
// rescaled) when it falls behind by more than 8 in log2 units: the weights stay below 2^8 and the sums exact enough,
// and after a row's first tiles it hardly ever happens.  The cap is monotonic, so the maximum is taken over raw scores.
// For scores well inside the cap tanh is its Taylor series, which costs fused multiply-adds on register pairs only; up to
// twice the cap it is the seventh convergent of Lambert's continued fraction (one reciprocal more per score); a warp
// whose tile has a larger score, or needs a mask, takes the general path.
//
// Sigmoid weights (nqb200_attention.sigmoid) need no maximum and no sum: a weight is 1 / (1 + 2^x), two weights share one
// reciprocal, 1 / a = b / (a b), with x clamped to 60 so that a b stays finite (weights below 2^-60 are 2^-60).
//
// Every wait is bounded; on expiry NQB200_ERR_WAIT_TIMEOUT goes to the status word, all roles drain and tensor memory is
// released.
#include "mixers.cuh"
#include "tma_utils.cuh"
#include "umma_utils.cuh"

namespace nqb200 {
namespace att {

constexpr int kTile = 128, kThreads = 384;
constexpr uint32_t kColS = 0, kColO = 256, kTmemCols = 512;
constexpr float kLog2e = 1.4426950408889634f, kLag = 8.f, kSeriesRange = 0.4f, kFractionRange = 2.f;

struct Params {
  nqb200_batch bt;
  bf16* out; int64_t out_stride;
  int heads, kv_heads, chunk;
  float scale, softcap, out_scale;
  const float* sink;
  int sigmoid; const float* temp; const float* bias;
  int* status;
};

constexpr uint32_t kSuspendNs = 20000;
__device__ __forceinline__ bool wait_bar(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* status) {
  const uint32_t b = smem_u32(bar);
  if (mbar_test_wait(b, parity)) return true;
  const unsigned long long t0 = global_timer_ns();
  for (;;) {
    if (mbar_try_wait_suspend(b, parity, kSuspendNs)) return true;
    if (*abort_flag) return false;
    if (global_timer_ns() - t0 > kWaitLimitNs) {
      *abort_flag = 1;
      if (status) atomicExch(status, NQB200_ERR_WAIT_TIMEOUT);
      return false;
    }
  }
}

// D[tmem] (+)= A[smem descriptor] * B[smem descriptor]; the descriptors' high halves are the same.
__device__ __forceinline__ void umma_ss_lohi(uint32_t d_tmem, uint32_t a_lo, uint32_t b_lo, uint32_t hi, uint32_t idesc, uint32_t accumulate) {
  asm volatile("{\n .reg .pred p;\n .reg .b64 a, b;\n setp.ne.b32 p, %5, 0;\n mov.b64 a, {%1, %3};\n mov.b64 b, {%2, %3};\n"
               " tcgen05.mma.cta_group::1.kind::f16 [%0], a, b, %4, p;\n}"
               ::"r"(d_tmem), "r"(a_lo), "r"(b_lo), "r"(hi), "r"(idesc), "r"(accumulate) : "memory");
}
// Operand whose rows in shared memory run along k (the contraction), 64 columns = 128 swizzled bytes a row: 8-row groups
// 1024 bytes apart along k, further blocks of 64 columns `block_bytes` apart.
__device__ __forceinline__ uint64_t smem_desc_mn(uint32_t addr, uint32_t block_bytes) {
  uint64_t d = 0;
  d |= (uint64_t)((addr & 0x3FFFFu) >> 4);
  d |= (uint64_t)(block_bytes >> 4) << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}
__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,"
               "%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
                 "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]),
                 "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]),
                 "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
               : "r"(taddr) : "memory");
}
__device__ __forceinline__ void tmem_st8(uint32_t taddr, const uint32_t (&r)[8]) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};"
               ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]) : "memory");
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
               ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
                 "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]) : "memory");
}
// pairs of floats in one 64-bit register
__device__ __forceinline__ uint64_t pair2(float lo, float hi) { uint64_t r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi)); return r; }
__device__ __forceinline__ void unpair2(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) { uint64_t r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) { uint64_t r; asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r;
}
__device__ __forceinline__ float max3(float a, float b, float c) { float r; asm("max.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c)); return r; }
__device__ __forceinline__ float min3(float a, float b, float c) { float r; asm("min.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c)); return r; }
__device__ __forceinline__ float ex2(float x) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}

template <int D, int V>
__global__ void __launch_bounds__(kThreads, 1)
attention_umma_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v,
                      const Params p) {
  constexpr uint32_t kQBytes = kTile * D * 2, kKBytes = kTile * D * 2, kVBytes = kTile * V * 2, kBox = kTile * 128;
  constexpr uint32_t kOffK = 2 * kQBytes, kOffV = kOffK + 2 * kKBytes;
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t bar_q, bar_kfull[2], bar_kfree[2], bar_vfull[2], bar_vfree[2], bar_s[2], bar_p[2][2], bar_pv[2], bar_o[2], bar_drain;
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort_i;
  volatile int* s_abort = &s_abort_i;
  const uint32_t smem = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  grid_launch_dependents();
  grid_dependency_wait();
  const int b = blockIdx.z, h = blockIdx.y, kvh = h / (p.heads / p.kv_heads);
  const int t0 = p.bt.cu[b], n = p.bt.cu[b + 1] - t0, pos0 = p.bt.pos0[b];
  const int i0 = (int)(gridDim.x - 1 - blockIdx.x) * 2 * kTile;     // long rows first
  if (i0 >= n) return;
  const int first = pos0 + i0, lo_first = p.chunk > 0 ? first / p.chunk * p.chunk : 0, kstart = lo_first / kTile * kTile;
  int nq[2];
#pragma unroll
  for (int q = 0; q < 2; ++q)
    nq[q] = i0 + q * kTile < n ? (pos0 + min(i0 + (q + 1) * kTile, n) - 1 - kstart) / kTile + 1 : 0;
  const int nmax = max(nq[0], nq[1]);

  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&bar_q), 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(smem_u32(&bar_kfull[s]), 1); mbar_init(smem_u32(&bar_kfree[s]), 1);
      mbar_init(smem_u32(&bar_vfull[s]), 1); mbar_init(smem_u32(&bar_vfree[s]), 1);
      mbar_init(smem_u32(&bar_s[s]), 1); mbar_init(smem_u32(&bar_p[s][0]), 4); mbar_init(smem_u32(&bar_p[s][1]), 4);
      mbar_init(smem_u32(&bar_pv[s]), 1); mbar_init(smem_u32(&bar_o[s]), 1);
    }
    mbar_init(smem_u32(&bar_drain), 1);
    s_abort_i = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(smem_u32(&s_tmem), kTmemCols); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = s_tmem;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA
    if (lane == 0) {
      prefetch_tmap(&tm_q); prefetch_tmap(&tm_k); prefetch_tmap(&tm_v);
      const int tiles_q = nq[1] > 0 ? 2 : 1;
      mbar_expect_tx(smem_u32(&bar_q), (uint32_t)tiles_q * kQBytes);
      for (int q = 0; q < tiles_q; ++q)
        for (int c = 0; c < D / 64; ++c) tma_load_2d(smem + q * kQBytes + c * kBox, &tm_q, h * D + c * 64, t0 + i0 + q * kTile, smem_u32(&bar_q));
      int issued = 0;
      for (int j = 0; j < nmax; ++j, ++issued) {
        const int s = j & 1, pos = kstart + j * kTile;
        if (j >= 2 && !wait_bar(&bar_kfree[s], ((j >> 1) - 1) & 1, s_abort, p.status)) break;
        const int row = (int)kv_row(p.bt, b, pos);    // the tile lies in one page
        mbar_expect_tx(smem_u32(&bar_kfull[s]), kKBytes);
        for (int c = 0; c < D / 64; ++c) tma_load_2d(smem + kOffK + s * kKBytes + c * kBox, &tm_k, kvh * D + c * 64, row, smem_u32(&bar_kfull[s]));
        if (j >= 2 && !wait_bar(&bar_vfree[s], ((j >> 1) - 1) & 1, s_abort, p.status)) {
          mbar_wait(smem_u32(&bar_kfull[s]), (j >> 1) & 1);
          break;
        }
        mbar_expect_tx(smem_u32(&bar_vfull[s]), kVBytes);
        for (int c = 0; c < V / 64; ++c) tma_load_2d(smem + kOffV + s * kVBytes + c * kBox, &tm_v, kvh * V + c * 64, row, smem_u32(&bar_vfull[s]));
      }
      // do not leave while a copy may still be landing
      mbar_wait(smem_u32(&bar_q), 0);
      for (int j = issued > 2 ? issued - 2 : 0; j < issued; ++j) {
        mbar_wait(smem_u32(&bar_kfull[j & 1]), (j >> 1) & 1);
        mbar_wait(smem_u32(&bar_vfull[j & 1]), (j >> 1) & 1);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA
    // One thread runs both tiles as two little state machines and never blocks on one of them: it polls for the first
    // and the second half of a tile's weights (then issues that half of O += P V) and for that product's end (P has been
    // read: then S of the next key tile may overwrite it).  A ring stage is handed back by whichever tile uses it second.
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc(1, 128, kTile);
      const uint32_t idesc_o = umma_idesc(1, 128, V) | (1u << 16);   // B's rows run along k
      const uint64_t dq = umma_smem_desc_sw128(smem), dk = umma_smem_desc_sw128(smem + kOffK), dv = smem_desc_mn(smem + kOffV, kBox);
      const uint32_t k_hi = (uint32_t)(dq >> 32), v_hi = (uint32_t)(dv >> 32), q_lo = (uint32_t)dq, k_lo = (uint32_t)dk, v_lo = (uint32_t)dv;
      auto scores = [&](int q, int s) {
        const uint32_t a = q_lo + q * (kQBytes >> 4), bk = k_lo + s * (kKBytes >> 4), d = tmem + kColS + q * 128;
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks)
          umma_ss_lohi(d, a + (ks >> 2) * (kBox >> 4) + (ks & 3) * 2, bk + (ks >> 2) * (kBox >> 4) + (ks & 3) * 2, k_hi, idesc_s, ks > 0 ? 1u : 0u);
        umma_commit(smem_u32(&bar_s[q]));
      };
      bool ok = wait_bar(&bar_q, 0, s_abort, p.status) && wait_bar(&bar_kfull[0], 0, s_abort, p.status);
      const int users = nq[1] > 0 ? 2 : 1;
      // tile of the next product; 0, 1: waits for that half of the weights, 2: for the product; users that have still to
      // issue on K / V tile j (by j & 1)
      int jq[2] = {0, 0};
      int phase[2] = {0, 0};
      auto users_of = [&](int j) { return users == 2 ? (j < nq[0]) + (j < nq[1]) : 1; };
      int kleft[2] = {0, users_of(1)}, vleft[2] = {users_of(0), users_of(1)};
      if (ok) {
        tc_fence_after();
        for (int q = 0; q < users; ++q) scores(q, 0);
        umma_commit(smem_u32(&bar_kfree[0]));
        kleft[0] = users_of(2);
      }
      unsigned long long t_last = global_timer_ns();
      uint32_t polls = 0;
      while (ok && (jq[0] < nq[0] || jq[1] < nq[1])) {
        bool moved = false;
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const int j = jq[q], s = j & 1, sn = s ^ 1;
          if (j >= nq[q]) continue;
          if (phase[q] < 2) {
            const int half = phase[q];
            if (!mbar_test_wait(smem_u32(&bar_p[q][half]), s) || !mbar_test_wait(smem_u32(&bar_vfull[s]), (j >> 1) & 1)) continue;
            tc_fence_after();
            const uint32_t d = tmem + kColO + q * 128, pa = tmem + kColS + q * 128 + half * 32, bv = v_lo + s * (kVBytes >> 4) + half * (8192 >> 4);
#pragma unroll
            for (int ks = 0; ks < kTile / 32; ++ks)
              umma_ts_lohi(d, pa + ks * 8, bv + ks * (2048 >> 4), v_hi, idesc_o, (j > 0 || half > 0 || ks > 0) ? 1u : 0u);
            phase[q] = half + 1;
            if (half == 1) {
              umma_commit(smem_u32(&bar_pv[q]));
              if (--vleft[s] == 0) { umma_commit(smem_u32(&bar_vfree[s])); vleft[s] = users_of(j + 2); }
              if (j == nq[q] - 1) { umma_commit(smem_u32(&bar_o[q])); jq[q] = j + 1; }
            }
          } else {
            if (!mbar_test_wait(smem_u32(&bar_pv[q]), s) || !mbar_test_wait(smem_u32(&bar_kfull[sn]), ((j + 1) >> 1) & 1)) continue;
            tc_fence_after();
            scores(q, sn);
            if (--kleft[sn] == 0) { umma_commit(smem_u32(&bar_kfree[sn])); kleft[sn] = users_of(j + 3); }
            jq[q] = j + 1;
            phase[q] = 0;
          }
          moved = true;
        }
        if (moved) {
          polls = 0;
        } else if ((++polls & 63u) == 0) {
          const unsigned long long now = global_timer_ns();
          if (polls == 64) t_last = now;
          if (*s_abort) ok = false;
          else if (now - t_last > kWaitLimitNs) {
            *s_abort = 1;
            if (p.status) atomicExch(p.status, NQB200_ERR_WAIT_TIMEOUT);
            ok = false;
          }
        }
      }
      // everything issued has completed before tensor memory may be released
      umma_commit(smem_u32(&bar_drain));
      mbar_wait(smem_u32(&bar_drain), 0);
    }
  } else if (warp >= 4) {
    // -------------------------------------------------------------- softmax
    const int q = (warp - 4) >> 2, quarter = warp & 3;
    const uint32_t tS = tmem + ((uint32_t)(32 * quarter) << 16) + kColS + q * 128, tO = tmem + ((uint32_t)(32 * quarter) << 16) + kColO + q * 128;
    const int i = i0 + q * kTile + quarter * 32 + lane, pos = pos0 + i, wfirst = pos - lane, wlast = wfirst + 31;
    const int lo = p.chunk > 0 ? pos / p.chunk * p.chunk : 0, lo_last = p.chunk > 0 ? wlast / p.chunk * p.chunk : 0;
    const bool capped = p.softcap > 0.f;
    const float ysc = capped ? p.scale / p.softcap : p.scale, top = capped ? p.softcap * kLog2e : kLog2e;
    auto score = [&](float s) {   // in log2 units
      const float y = s * ysc;
      return top * (capped ? tanh_fast(y) : y);
    };
    const uint64_t ysc2 = pair2(ysc, ysc), k1 = pair2(top, top), k3 = pair2(-top / 3.f, -top / 3.f), k5 = pair2(top * (2.f / 15.f), top * (2.f / 15.f)),
                   k7 = pair2(-top * (17.f / 315.f), -top * (17.f / 315.f)), k9 = pair2(top * (62.f / 2835.f), top * (62.f / 2835.f));
    auto half_done = [&](int half) {   // that half of the weights is in tensor memory
      tc_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&bar_p[q][half]));
    };
    const float sg_scale = -p.scale * (p.temp ? p.temp[h] : 1.f) * kLog2e, sg_shift = p.bias ? -p.bias[h] * kLog2e : 0.f;
    const uint64_t sg_scale2 = pair2(sg_scale, sg_scale), sg_shift2 = pair2(sg_shift, sg_shift), one2 = pair2(1.f, 1.f);
    auto sigmoid2 = [&](uint32_t s0, uint32_t s1, float& w0, float& w1) {
      float x0, x1;
      unpair2(fma2(pair2(__uint_as_float(s0), __uint_as_float(s1)), sg_scale2, sg_shift2), x0, x1);
      float d0, d1;
      unpair2(add2(pair2(ex2(fminf(x0, 60.f)), ex2(fminf(x1, 60.f))), one2), d0, d1);
      const float r = rcp_fast(d0 * d1);
      w0 = r * d1;
      w1 = r * d0;
    };
    const float sink = p.sink ? p.sink[h] * kLog2e : -INFINITY;
    float m = sink, l = 0.f;
    uint64_t lsum = pair2(0.f, 0.f);
    bool ok = true;
    for (int j = 0; j < nq[q]; ++j) {
      ok = wait_bar(&bar_s[q], j & 1, s_abort, p.status);
      if (!__all_sync(0xFFFFFFFFu, ok)) { ok = false; break; }
      tc_fence_after();
      const int key0 = kstart + j * kTile;
      const bool masked = key0 + kTile - 1 > wfirst || key0 < lo_last;     // for any row of the warp
      uint32_t r[4][32];     // the row's scores, all of them
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld32(tS + c * 32, r[c]);
      tc_wait_ld();
      if (p.sigmoid) {
        if (!masked) {
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            uint32_t w[16];
#pragma unroll
            for (int e = 0; e < 16; ++e) {
              float x0, x1;
              sigmoid2(r[c][2 * e], r[c][2 * e + 1], x0, x1);
              w[e] = pack_bf16(x0, x1);
            }
            tmem_st16(tS + c * 16, w);
            if (c == 1) half_done(0);
          }
        } else {
#pragma unroll 1
          for (int c = 0; c < 8; ++c) {
            uint32_t v[16], w[8];
            tmem_ld_32x32b_x16(tS + c * 16, v);
            tc_wait_ld();
#pragma unroll
            for (int e = 0; e < 8; ++e) {
              const int key = key0 + c * 16 + 2 * e;
              float x0, x1;
              sigmoid2(v[2 * e], v[2 * e + 1], x0, x1);
              w[e] = pack_bf16(key <= pos && key >= lo ? x0 : 0.f, key + 1 <= pos && key + 1 >= lo ? x1 : 0.f);
            }
            tmem_st8(tS + c * 8, w);      // lies behind what has been read of S
            if (c == 3) half_done(0);
          }
        }
        half_done(1);
        continue;
      }
      float mx = -INFINITY, ab = 0.f;
      if (!masked) {
        float hi[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY}, lw[4] = {INFINITY, INFINITY, INFINITY, INFINITY};
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int e = 0; e < 32; e += 2) {
            const int k = (e >> 1) & 3;
            hi[k] = max3(hi[k], __uint_as_float(r[c][e]), __uint_as_float(r[c][e + 1]));
            lw[k] = min3(lw[k], __uint_as_float(r[c][e]), __uint_as_float(r[c][e + 1]));
          }
        mx = fmaxf(fmaxf(hi[0], hi[1]), fmaxf(hi[2], hi[3]));
        ab = fmaxf(mx, -fminf(fminf(lw[0], lw[1]), fminf(lw[2], lw[3])));
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int e = 0; e < 32; ++e) {
            const int key = key0 + c * 32 + e;
            mx = (key <= pos && key >= lo) ? fmaxf(mx, __uint_as_float(r[c][e])) : mx;
          }
      }
      const float mt = mx == -INFINITY ? mx : score(mx), mn = fmaxf(m, mt);
      if (j == 0) {
        l = p.sink ? ex2(sink - mn) : 0.f;
        m = mn;
      } else {
        const bool move = mn > m + kLag;      // also from -inf
        if (__any_sync(0xFFFFFFFFu, move)) {
          const float f = move ? ex2(m - mn) : 1.f;
          m = move ? mn : m;
          l *= f;
          float a, c2;
          unpair2(lsum, a, c2);
          lsum = pair2(a * f, c2 * f);
#pragma unroll 1
          for (int c = 0; c < V / 8; ++c) {   // rare: small pieces, few registers
            uint32_t o[8];
            tmem_ld_32x32b_x8(tO + c * 8, o);
            tc_wait_ld();
#pragma unroll
            for (int e = 0; e < 8; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * f);
            tmem_st8(tO + c * 8, o);
          }
          tc_wait_st();
        }
      }
      const float mu = m == -INFINITY ? 0.f : m;
      const int range = masked ? 2 : !capped || __all_sync(0xFFFFFFFFu, ab * ysc <= kSeriesRange) ? 0 : __all_sync(0xFFFFFFFFu, ab * ysc <= kFractionRange) ? 1 : 2;
      if (range == 1) {
        // tanh y = y (10395 + 1260 y^2 + 21 y^4) / (10395 + 4725 y^2 + 210 y^4 + y^6)
        const uint64_t n0 = pair2(10395.f, 10395.f), n1 = pair2(1260.f, 1260.f), n2 = pair2(21.f, 21.f), d1 = pair2(4725.f, 4725.f), d2 = pair2(210.f, 210.f),
                       nm2 = pair2(-mu, -mu);
        uint64_t ls[2] = {lsum, 0};
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t w[16];
#pragma unroll
          for (int e = 0; e < 16; ++e) {
            const uint64_t y = mul2(pair2(__uint_as_float(r[c][2 * e]), __uint_as_float(r[c][2 * e + 1])), ysc2), y2 = mul2(y, y);
            const uint64_t num = mul2(mul2(y, k1), fma2(fma2(n2, y2, n1), y2, n0)), den = fma2(fma2(add2(y2, d2), y2, d1), y2, n0);
            float a, c2, x0, x1;
            unpair2(den, a, c2);
            unpair2(fma2(num, pair2(rcp_fast(a), rcp_fast(c2)), nm2), x0, x1);
            x0 = ex2(x0);
            x1 = ex2(x1);
            ls[e & 1] = add2(ls[e & 1], pair2(x0, x1));
            w[e] = pack_bf16(x0, x1);
          }
          tmem_st16(tS + c * 16, w);
          if (c == 1) half_done(0);
        }
        lsum = add2(ls[0], ls[1]);
      } else if (range == 0) {
        const uint64_t nm2 = pair2(-mu, -mu);
        uint64_t ls[4] = {lsum, 0, 0, 0};
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t w[16];
#pragma unroll
          for (int e = 0; e < 16; ++e) {
            const uint64_t y = mul2(pair2(__uint_as_float(r[c][2 * e]), __uint_as_float(r[c][2 * e + 1])), ysc2);
            uint64_t arg;
            if (capped) {
              const uint64_t y2 = mul2(y, y);
              arg = fma2(y, fma2(fma2(fma2(fma2(k9, y2, k7), y2, k5), y2, k3), y2, k1), nm2);
            } else {
              arg = fma2(y, k1, nm2);
            }
            float x0, x1;
            unpair2(arg, x0, x1);
            x0 = ex2(x0);
            x1 = ex2(x1);
            ls[e & 3] = add2(ls[e & 3], pair2(x0, x1));
            w[e] = pack_bf16(x0, x1);
          }
          tmem_st16(tS + c * 16, w);
          if (c == 1) half_done(0);
        }
        lsum = add2(add2(ls[0], ls[1]), add2(ls[2], ls[3]));
      } else {
        // from tensor memory again, a piece at a time: compact code for the few tiles at the edges
#pragma unroll 1
        for (int c = 0; c < 8; ++c) {
          uint32_t v[16], w[8];
          tmem_ld_32x32b_x16(tS + c * 16, v);
          tc_wait_ld();
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            float x[2];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              const int key = key0 + c * 16 + 2 * e + u;
              x[u] = (key <= pos && key >= lo) ? ex2(score(__uint_as_float(v[2 * e + u])) - mu) : 0.f;
            }
            lsum = add2(lsum, pair2(x[0], x[1]));
            w[e] = pack_bf16(x[0], x[1]);
          }
          tmem_st8(tS + c * 8, w);      // lies behind what has been read of S
          if (c == 3) half_done(0);
        }
      }
      half_done(1);
    }
    if (ok && nq[q] > 0) {
      ok = wait_bar(&bar_o[q], 0, s_abort, p.status);
      if (__all_sync(0xFFFFFFFFu, ok)) {
        tc_fence_after();
        float a, c2;
        unpair2(lsum, a, c2);
        const float f = p.sigmoid ? p.out_scale : p.out_scale / (l + a + c2);
        bf16* dst = p.out + (size_t)(t0 + i) * p.out_stride + (size_t)h * V;
#pragma unroll
        for (int c = 0; c < V / 32; ++c) {
          uint32_t r[32];
          tmem_ld32(tO + c * 32, r);
          tc_wait_ld();
          if (i < n) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              uint4 v;
              v.x = pack_bf16(__uint_as_float(r[8 * e]) * f, __uint_as_float(r[8 * e + 1]) * f);
              v.y = pack_bf16(__uint_as_float(r[8 * e + 2]) * f, __uint_as_float(r[8 * e + 3]) * f);
              v.z = pack_bf16(__uint_as_float(r[8 * e + 4]) * f, __uint_as_float(r[8 * e + 5]) * f);
              v.w = pack_bf16(__uint_as_float(r[8 * e + 6]) * f, __uint_as_float(r[8 * e + 7]) * f);
              *reinterpret_cast<uint4*>(dst + c * 32 + e * 8) = v;
            }
          }
          __syncwarp();
        }
        tc_fence_before();
      }
    }
  }
  // all roles meet here, also after a give-up, so that tensor memory is always released
  tc_fence_before();
  __syncthreads();
  if (warp == 1) { __syncwarp(); tc_fence_after(); tmem_dealloc(tmem, kTmemCols); }
}

static bool encode_rows(CUtensorMap* m, const void* base, uint64_t rows, uint64_t cols, uint64_t row_bytes) {
  PFN_cuTensorMapEncodeTiled enc = tensor_map_encoder();
  if (!enc) return false;
  cuuint64_t dims[2] = {cols, rows}, strides[1] = {row_bytes};
  cuuint32_t box[2] = {64, (cuuint32_t)kTile}, estr[2] = {1, 1};
  return enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int D, int V>
static int launch(const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& v, const Params& p, cudaStream_t st) {
  // at least 120 KB, whatever the sizes: one CTA per SM, because a CTA takes all of the SM's tensor memory
  const size_t need = (size_t)kTile * (2 * D + 2 * D + 2 * V) * 2 + 1024, smem = need > 120 * 1024 ? need : 120 * 1024;
  if (cudaFuncSetAttribute(attention_umma_kernel<D, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return NQB200_ERR_LAUNCH;
  }
  const dim3 grid((unsigned)((p.bt.max_len + 2 * kTile - 1) / (2 * kTile)), (unsigned)p.heads, (unsigned)p.bt.batch);
  return launch_overlapped(attention_umma_kernel<D, V>, grid, dim3(kThreads), smem, st, q, k, v, p);
}

}  // namespace att

// From 128 tokens and, with chunks, 512 positions a chunk: below, tiles of 128 x 256 are mostly mask.
bool attention_umma_supports(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, const void* out, int64_t out_stride,
                             int64_t cache_rows, const nqb200_attention* a, const nqb200_batch* b) {
  return (a->dim == 64 || a->dim == 128) && (a->vdim == 64 || a->vdim == 128) && b->block_size % att::kTile == 0 && cache_rows > 0 &&
         cache_rows % b->block_size == 0 && b->max_len >= att::kTile && (a->chunk <= 0 || a->chunk >= 512) && a->scale > 0.f && q_stride % 8 == 0 &&
         out_stride % 8 == 0 && aligned16(q) && aligned16(k_cache) && aligned16(v_cache) && aligned16(out);
}
int attention_umma(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, void* out, int64_t out_stride, int64_t cache_rows,
                   const nqb200_attention* a, const nqb200_batch* b, int* status, cudaStream_t st) {
  CUtensorMap tq, tk, tv;
  if (!att::encode_rows(&tq, q, b->tokens, (uint64_t)a->heads * a->dim, (uint64_t)q_stride * 2) ||
      !att::encode_rows(&tk, k_cache, cache_rows, (uint64_t)a->kv_heads * a->dim, (uint64_t)a->kv_heads * a->dim * 2) ||
      !att::encode_rows(&tv, v_cache, cache_rows, (uint64_t)a->kv_heads * a->vdim, (uint64_t)a->kv_heads * a->vdim * 2))
    return NQB200_ERR_LAUNCH;
  att::Params p = {};
  p.bt = *b; p.out = (bf16*)out; p.out_stride = out_stride; p.heads = a->heads; p.kv_heads = a->kv_heads; p.chunk = a->chunk;
  p.scale = a->scale; p.softcap = a->softcap; p.out_scale = a->out_scale; p.sink = a->sink; p.sigmoid = a->sigmoid; p.temp = a->temp; p.bias = a->bias;
  p.status = status;
  if (a->dim == 64) return a->vdim == 64 ? att::launch<64, 64>(tq, tk, tv, p, st) : att::launch<64, 128>(tq, tk, tv, p, st);
  return a->vdim == 64 ? att::launch<128, 64>(tq, tk, tv, p, st) : att::launch<128, 128>(tq, tk, tv, p, st);
}

}  // namespace nqb200
