// The experts' linears of steps with more than a decode step's tokens, on the 5th-generation tensor cores: a grouped GEMM
// whose groups (the pairs of every expert) are read from the plan on the device.
//
//   D[feature, pair] (tensor memory, fp32) = sum_k w[expert][feature, k] x[row(pair), k]
//
// The two CTAs of a cluster work as one (tcgen05.mma.cta_group::2): 256 features, 128 from each CTA's shared memory, by up to
// 256 pairs of one expert, of which each CTA loads half.  Pairs are the MMA's N, in steps of 32, so that an expert's last
// tile costs what it holds and a step of few tokens streams the weights past a narrow tile.  The tiles of all experts are
// numbered, feature tiles fastest (they share the pairs' rows), and dealt to the persistent clusters in turn.
//
//   warp 0        TMA: the weight tile, and for the second linear the pairs' rows, which are contiguous.  A ring of five
//                 stages of 64 k.
//   warp 1        the leader's: one thread issues the MMAs; the other CTA's: reports its landed stages to the leader.
//   warps 2-9     epilogue: accumulator (two of them take turns) -> gelu or the pair's weight -> 16 bits in shared memory,
//                 [pair][feature] -> rows of 256 bytes to their places in the output.
//   warps 10-13   first linear: the pairs' rows, gathered by token with cp.async into the swizzled layout, two stages ahead
//                 of what they report (TMA's gather of four rows per instruction took 1.4 us per stage of 128 rows).
//
// Every wait is bounded; on expiry NQB200_ERR_WAIT_TIMEOUT goes to the status word, all roles drain and tensor memory is
// released.
#include "moe.cuh"
#include "tma_utils.cuh"
#include "umma_utils.cuh"

namespace nqb200 {
namespace moe {

constexpr int kStages = 5, kEpiWarps = 8, kLoadWarps = 4, kMaxExperts = 1024;
constexpr int kTile = 256, kStepK = 64;
constexpr int kABytes = 128 * kStepK * 2, kStageBytes = 2 * kABytes;
constexpr int kOffOut = kStages * kStageBytes, kRound = 128, kOutBytes = kRound * 128 * 2;
constexpr int kSmem = kOffOut + kOutBytes + 1024;
constexpr int kTmemCols = 512;
constexpr int kAhead = 2;   // stages between a gather and its report

struct Params {
  const int32_t* offsets; const int32_t* order; const float* weight;
  const bf16* x; bf16* out;
  int N, K, experts, top, ntn, steps, clusters;
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
// One arrival on the barrier at this offset in both CTAs when every MMA issued so far by this thread has completed.
__device__ __forceinline__ void commit_both(uint32_t bar) {
  asm volatile("tcgen05.commit.cta_group::2.mbarrier::arrive::one.shared::cluster.multicast::cluster.b64 [%0], %1;"
               ::"r"(bar), "h"((uint16_t)3) : "memory");
}
// Both operands in shared memory, M = 256 over the pair; the descriptors' high halves are the same.
__device__ __forceinline__ void umma_ss_pair(uint32_t d_tmem, uint32_t a_lo, uint32_t b_lo, uint32_t hi, uint32_t idesc, uint32_t accumulate) {
  asm volatile("{\n .reg .pred p;\n .reg .b64 a, b;\n setp.ne.b32 p, %5, 0;\n mov.b64 a, {%1, %3};\n mov.b64 b, {%2, %3};\n"
               " tcgen05.mma.cta_group::2.kind::f16 [%0], a, b, %4, p;\n}"
               ::"r"(d_tmem), "r"(a_lo), "r"(b_lo), "r"(hi), "r"(idesc), "r"(accumulate) : "memory");
}
__device__ __forceinline__ void copy16(uint32_t dst, const void* src, bool ok) {   // zeros where not ok
  const int n = ok ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n));
}
// Barrier of the epilogue's threads that tells all of them whether all of them are well.
__device__ __forceinline__ bool epi_all(bool ok) {
  uint32_t r;
  asm volatile("{\n .reg .pred p, q;\n setp.ne.b32 p, %1, 0;\n barrier.cta.red.and.pred q, 1, %2, p;\n selp.u32 %0, 1, 0, q;\n}"
               : "=r"(r) : "r"((uint32_t)ok), "r"((uint32_t)(kEpiWarps * 32)) : "memory");
  return r != 0;
}

struct Item { int expert, feature, lo, cnt, nt; };   // first feature; first pair, pairs, and pairs rounded up to the MMA's steps
__device__ __forceinline__ Item locate(const Params& p, const int* tiles, int item) {   // tiles: running count of pair tiles up to each expert
  const int tg = item / p.ntn;
  int a = 0, b = p.experts - 1;
  while (a < b) {
    const int m = (a + b) >> 1;
    if (tiles[m] > tg) b = m; else a = m + 1;
  }
  const int before = a > 0 ? tiles[a - 1] : 0, n = tiles[a] - before, j = tg - before;
  const int first = p.offsets[a], c = p.offsets[a + 1] - first, per = ((c + n - 1) / n + 31) & ~31;
  Item it;
  it.expert = a;
  it.feature = (item - tg * p.ntn) * kTile;
  it.lo = first + j * per;
  it.cnt = min(per, c - j * per);
  it.nt = (it.cnt + 31) & ~31;
  return it;
}

template <bool UP>
__global__ void __launch_bounds__((2 + kEpiWarps + (UP ? kLoadWarps : 0)) * 32, 1) moe_umma_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x, const __grid_constant__ CUtensorMap tm_x128,
                const Params p) {
  constexpr int kThreads = (2 + kEpiWarps + (UP ? kLoadWarps : 0)) * 32, kLocal = 1 + (UP ? kLoadWarps : 0);
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t bar_full[kStages], bar_free[kStages], bar_dfull[2], bar_dempty[2], bar_drain;
  __shared__ int tiles[kMaxExperts], s_rows[2][kTile];
  __shared__ float s_weight[2][kTile];
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort_i;
  volatile int* s_abort = &s_abort_i;
  const uint32_t smem = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, cluster = blockIdx.x >> 1;
  const uint32_t rank = cluster_ctarank();

  grid_launch_dependents();
  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) {
      // the leader's stage is complete when its own copies have landed and the other CTA has reported its own
      mbar_init(smem_u32(&bar_full[s]), kLocal + (rank == 0 ? 1 : 0));
      mbar_init(smem_u32(&bar_free[s]), 1);
    }
    for (int d = 0; d < 2; ++d) { mbar_init(smem_u32(&bar_dfull[d]), 1); mbar_init(smem_u32(&bar_dempty[d]), 2 * kEpiWarps); }
    mbar_init(smem_u32(&bar_drain), 1);
    s_abort_i = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc_pair(smem_u32(&s_tmem), kTmemCols); tmem_relinquish_pair(); }
  grid_dependency_wait();
  for (int e = threadIdx.x; e < p.experts; e += kThreads) tiles[e] = (p.offsets[e + 1] - p.offsets[e] + kTile - 1) / kTile;
  __syncthreads();
  if (warp == 0) {   // running sum: a lane sums a run of experts, the warp the runs
    const int per = (p.experts + 31) / 32, e0 = min(lane * per, p.experts), e1 = min(e0 + per, p.experts);
    int sum = 0;
    for (int e = e0; e < e1; ++e) sum += tiles[e];
    int run = sum;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int u = __shfl_up_sync(0xFFFFFFFFu, run, o);
      if (lane >= o) run += u;
    }
    run -= sum;
    for (int e = e0; e < e1; ++e) { run += tiles[e]; tiles[e] = run; }
  }
  tc_fence_before();
  __syncthreads();
  cluster_sync_all();  // both CTAs' barriers exist before anything arrives on them from the other side
  tc_fence_after();
  const uint32_t tmem = s_tmem;
  const int items = tiles[p.experts - 1] * p.ntn;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA
    if (lane == 0) { prefetch_tmap(&tm_w); prefetch_tmap(&tm_x); prefetch_tmap(&tm_x128); }
    int n = 0;            // stages filled so far
    bool ok = true;
    for (int item = cluster; ok && item < items; item += p.clusters) {
      const Item it = locate(p, tiles, item);
      const int th = it.nt / 2, w_row = it.expert * p.N + it.feature + (int)rank * 128, first = (int)rank * th;
      // one box of 128 rows where that is not far too many (what lies behind the tile is not used): boxes cost by the piece
      const bool one = th > 48;
      const uint32_t bytes = (uint32_t)kABytes + (UP ? 0u : one ? 128u * 128u : (uint32_t)th * 128u);
      for (int k = 0; k < p.steps; ++k, ++n) {
        const int s = n % kStages;
        const uint32_t st = smem + s * kStageBytes, bar = smem_u32(&bar_full[s]);
        if (lane == 0) {
          if (n >= kStages) ok = wait_bar(&bar_free[s], ((n / kStages) - 1) & 1, s_abort, p.status);
          if (ok) mbar_expect_tx(bar, bytes);
        }
        ok = __shfl_sync(0xFFFFFFFFu, (int)ok, 0) != 0;
        if (!ok) break;
        if (lane == 0) tma_load_2d(st, &tm_w, k * kStepK, w_row, bar);
        if (!UP && one && lane == 0) tma_load_2d(st + kABytes, &tm_x128, k * kStepK, it.lo + first, bar);
        if (!UP && !one && 16 * lane < th) tma_load_2d(st + kABytes + lane * 2048, &tm_x, k * kStepK, it.lo + first + 16 * lane, bar);
      }
    }
    // do not leave while a copy may still be landing
    __syncwarp();
    if (lane == 0)
      for (int j = n > kStages ? n - kStages : 0; j < n; ++j) mbar_wait(smem_u32(&bar_full[j % kStages]), (j / kStages) & 1);
  } else if (warp == 1) {
    if (lane == 0 && rank == 0) {
      // ---------------------------------------------------------------- MMA
      const uint64_t desc = umma_smem_desc_sw128(smem);
      const uint32_t hi = (uint32_t)(desc >> 32), lo0 = (uint32_t)desc;
      int s = 0, li = 0;
      uint32_t phase = 0;
      bool ok = true;
      for (int item = cluster; ok && item < items; item += p.clusters, ++li) {
        const Item it = locate(p, tiles, item);
        const uint32_t idesc = umma_idesc(1, 256, it.nt), d = tmem + (li & 1) * 256;
        if (li >= 2 && !wait_bar(&bar_dempty[li & 1], ((li >> 1) - 1) & 1, s_abort, p.status)) { ok = false; break; }
        for (int k = 0; k < p.steps; ++k) {
          if (!wait_bar(&bar_full[s], phase, s_abort, p.status)) { ok = false; break; }
          tc_fence_after();
          const uint32_t a = lo0 + s * (kStageBytes >> 4), b = a + (kABytes >> 4);
#pragma unroll
          for (int ks = 0; ks < kStepK / 16; ++ks) umma_ss_pair(d, a + ks * 2, b + ks * 2, hi, idesc, (k | ks) != 0 ? 1u : 0u);
          commit_both(smem_u32(&bar_free[s]));
          if (++s == kStages) { s = 0; phase ^= 1u; }
        }
        if (ok) commit_both(smem_u32(&bar_dfull[li & 1]));
      }
      // everything issued has completed before tensor memory may be released
      umma_commit_pair(map_to_cta(smem_u32(&bar_drain), 0));
      mbar_wait(smem_u32(&bar_drain), 0);
    } else if (lane == 0) {
      // -------------------------------------------- the other CTA's stages
      int s = 0;
      uint32_t phase = 0;
      bool ok = true;
      const uint32_t leader = map_to_cta(smem_u32(&bar_full[0]), 0);
      for (int item = cluster; ok && item < items; item += p.clusters)
        for (int k = 0; k < p.steps; ++k) {
          if (!wait_bar(&bar_full[s], phase, s_abort, p.status)) { ok = false; break; }
          mbar_arrive_cluster(leader + (uint32_t)s * 8u);
          if (++s == kStages) { s = 0; phase ^= 1u; }
        }
    }
  } else if (UP && warp >= 2 + kEpiWarps) {
    // ------------------------------------------------------------ gathered rows
    const int t = threadIdx.x - (2 + kEpiWarps) * 32, chunk = t & 7, row0 = t >> 3;
    const uint32_t dst0 = smem + kABytes + row0 * 128 + ((chunk ^ (row0 & 7)) << 4);   // rows 16 apart keep the same swizzle
    int n = 0;
    bool ok = true;
    auto report = [&](int m) {   // copies of stage m have landed: the tensor core reads them through the async proxy
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&bar_full[m % kStages]));
    };
    for (int item = cluster; ok && item < items; item += p.clusters) {
      const Item it = locate(p, tiles, item);
      const int th = it.nt / 2, first = (int)rank * th;
      const bf16* src[8];
#pragma unroll
      for (int i = 0; i < 8; ++i)
        src[i] = p.x + (size_t)(p.order[it.lo + min(first + row0 + 16 * i, it.cnt - 1)] / p.top) * p.K + chunk * 8;
      for (int k = 0; k < p.steps; ++k, ++n) {
        const int s = n % kStages;
        if (n >= kStages) ok = wait_bar(&bar_free[s], ((n / kStages) - 1) & 1, s_abort, p.status);
        ok = __all_sync(0xFFFFFFFFu, ok) != 0;
        if (!ok) break;
        const bool in = k * kStepK + chunk * 8 < p.K;   // K is a multiple of 8
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (16 * i < th) copy16(dst0 + s * kStageBytes + i * 2048, in ? src[i] + k * kStepK : src[i], in);
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (n >= kAhead) {
          asm volatile("cp.async.wait_group %0;" ::"n"(kAhead) : "memory");
          report(n - kAhead);
        }
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    for (int m = n > kAhead ? n - kAhead : 0; m < n; ++m) report(m);
  } else {
    // -------------------------------------------------------------- epilogue
    const int quarter = warp & 3, half = (warp - 2) >> 2, tid = threadIdx.x - 64;
    const uint32_t lanes = tmem + ((uint32_t)(32 * quarter) << 16);
    uint8_t* stage = smem_raw + (smem - smem_u32(smem_raw)) + kOffOut;
    int li = 0;
    for (int item = cluster; item < items; item += p.clusters, ++li) {
      const Item it = locate(p, tiles, item);
      const int buf = li & 1;
      if (tid < it.cnt) {   // where pair `tid` of the tile goes, and its weight
        const int pair = UP ? it.lo + tid : p.order[it.lo + tid];
        s_rows[buf][tid] = pair;
        s_weight[buf][tid] = UP ? 1.f : p.weight[pair];
      }
      const bool ok = wait_bar(&bar_dfull[buf], (li >> 1) & 1, s_abort, p.status);
      if (!epi_all(ok)) break;
      tc_fence_after();
      const int n0 = it.feature + (int)rank * 128;
      for (int c0 = 0; c0 < it.nt; c0 += kRound) {
        const int end = min(c0 + kRound, it.nt);
        if (c0 > 0) epi_all(true);    // the round before has been stored
        for (int c = c0 + 16 * half; c < end; c += 32) {
          uint32_t d[16];
          tmem_ld_32x32b_x16(lanes + buf * 256 + c, d);
          tc_wait_ld();
          uint8_t* dst = stage + (size_t)(c - c0) * 256 + (quarter * 32 + lane) * 2;
          if (UP) {
#pragma unroll
            for (int i = 0; i < 16; ++i) *reinterpret_cast<bf16*>(dst + i * 256) = __float2bfloat16_rn(gelu_erf_f(__uint_as_float(d[i])));
          } else {
#pragma unroll
            for (int i = 0; i < 16; ++i) *reinterpret_cast<bf16*>(dst + i * 256) = __float2bfloat16_rn(__uint_as_float(d[i]) * s_weight[buf][c + i]);
          }
        }
        if (end == it.nt) {           // the accumulator has been read
          tc_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive_cluster(map_to_cta(smem_u32(&bar_dempty[buf]), 0));
        }
        epi_all(true);
        const int n = n0 + (tid & 15) * 8, last = min(end, it.cnt);
        if (n < p.N)
          for (int r = c0 + (tid >> 4); r < last; r += 16)
            *reinterpret_cast<uint4*>(p.out + (size_t)s_rows[buf][r] * p.N + n) = *reinterpret_cast<const uint4*>(stage + (size_t)(r - c0) * 256 + (tid & 15) * 16);
      }
      epi_all(true);                  // before the next tile is staged
    }
  }
  // all roles of both CTAs meet here, also after a give-up: neither may leave while the other can still read its shared
  // or tensor memory or arrive on its barriers
  tc_fence_before();
  __syncthreads();
  cluster_sync_all();
  if (warp == 1) { __syncwarp(); tc_fence_after(); tmem_dealloc_pair(tmem, kTmemCols); }
}

}  // namespace moe

bool moe_umma_supports(int64_t tokens, int64_t N, int64_t K, int64_t top) {
  return tokens > 0 && K % 8 == 0 && K >= moe::kStepK && N % 8 == 0 && N >= 32 && tokens * top <= (1 << 30);
}

int moe_umma(const MoeArgs& a) {
  using namespace moe;
  if (a.experts > kMaxExperts) return NQB200_ERR_TOO_LARGE;
  alignas(64) CUtensorMap tw, tx, txl;
  const int64_t pairs = (int64_t)a.tokens * a.top;
  const bool up = a.kind == NQB200_MOE_UP;
  bool ok = encode_2d(&tw, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.w, (uint64_t)a.experts * a.N, a.K, 128, kStepK, CU_TENSOR_MAP_SWIZZLE_128B);
  ok = ok && encode_2d(&tx, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.x, up ? a.tokens : pairs, a.K, 16, kStepK, CU_TENSOR_MAP_SWIZZLE_128B);   // second linear
  ok = ok && encode_2d(&txl, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.x, up ? a.tokens : pairs, a.K, 128, kStepK, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!ok) return NQB200_ERR_LAUNCH;
  Params p = {};
  p.offsets = a.plan.offsets; p.order = a.plan.order; p.weight = a.plan.weight; p.x = (const bf16*)a.x; p.out = (bf16*)a.out;
  p.N = a.N; p.K = a.K; p.experts = a.experts; p.top = a.top;
  p.ntn = (a.N + kTile - 1) / kTile; p.steps = (a.K + kStepK - 1) / kStepK; p.status = a.status;
  const int64_t most = ((pairs < a.experts ? pairs : a.experts) + pairs / kTile) * p.ntn;
  p.clusters = (int)(most < kNumSMs / 2 ? most : kNumSMs / 2);
  auto kernel = up ? moe_umma_kernel<true> : moe_umma_kernel<false>;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem) != cudaSuccess) { cudaGetLastError(); return NQB200_ERR_LAUNCH; }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)(2 * p.clusters)); cfg.blockDim = dim3((2 + kEpiWarps + (up ? kLoadWarps : 0)) * 32); cfg.dynamicSmemBytes = kSmem; cfg.stream = a.stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = 2; attr[1].val.clusterDim.y = 1; attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr; cfg.numAttrs = 2;
  if (cudaLaunchKernelEx(&cfg, kernel, tw, tx, txl, p) != cudaSuccess) { cudaGetLastError(); return NQB200_ERR_LAUNCH; }
  return NQB200_OK;
}

}  // namespace nqb200
