// bf16 projection on the 5th-generation tensor cores for 3 rows and more: y = epilogue(x W^T + b), any N and K.
//
// The scheme of gemm_tc.cu on bf16 operands: A = 128 weight rows x 64 k, B = TN activation rows x 64 k, both K-major and
// brought into 128-byte swizzled shared memory by TMA, D = 128 x TN fp32 in tensor memory; warp 0 issues the loads, warp 1
// the MMAs, the others run the epilogue; split-K over a thread-block cluster with the partial accumulators collected in
// rank 0's shared memory.  Row strides are free (multiples of 8 elements), and ragged N, K and M edges read as zeros
// through the tensor maps, so no shape needs another kernel.  Weights are parameters: their first tiles are requested
// before the dependency wait.  No cluster multicast; every mbarrier wait is bounded (JG_ETIMEDOUT at the next
// synchronisation).
#include <stdlib.h>

#include "dense.cuh"
#include "tcgen05.cuh"

constexpr int DT_BM = 128, DT_BK = 64;

struct DtArgs {
  bf16* y;
  float* y32;
  const float *b0, *b1;
  int* err;
  int M, N, K, ldy, w_late;
  float limit;
  DenseOut out;
};

template <int TN, bool GLU, bool HALF>
struct DtCfg {
  static constexpr int NW = GLU ? 2 : 1;
  static constexpr int NCOL = NW * TN;
  static constexpr int EPW = TN >= 128 ? 4 : 2;  // epilogue warps per 32-lane quarter
  static constexpr int THREADS = 64 + 128 * EPW;
  static constexpr uint32_t A_BYTES = DT_BM * DT_BK * 2, B_BYTES = TN * DT_BK * 2, STAGE_BYTES = NW * A_BYTES + B_BYTES;
  static constexpr int STAGES_FIT = ((HALF ? 110 : 225) * 1024) / STAGE_BYTES;
  static constexpr int STAGES = STAGES_FIT > 10 ? 10 : STAGES_FIT;
  static constexpr uint32_t TMEM_COLS = NCOL <= 32 ? 32 : (NCOL <= 64 ? 64 : (NCOL <= 128 ? 128 : (NCOL <= 256 ? 256 : 512)));
  static constexpr size_t SMEM = (size_t)STAGES * STAGE_BYTES + 1024;
  static constexpr int MAX_KS = 1 + (int)(((size_t)STAGES * STAGE_BYTES) / ((size_t)NCOL * DT_BM * 4));
};

template <int TN, bool GLU, bool HALF>
__global__ void __launch_bounds__(DtCfg<TN, GLU, HALF>::THREADS, HALF ? 2 : 1)
    dense_tc_kernel(const __grid_constant__ CUtensorMap tm_w0, const __grid_constant__ CUtensorMap tm_w1, const __grid_constant__ CUtensorMap tm_x, const DtArgs a) {
  using Cfg = DtCfg<TN, GLU, HALF>;
  constexpr int NW = Cfg::NW, STAGES = Cfg::STAGES, NCOL = Cfg::NCOL;
  constexpr uint32_t A_BYTES = Cfg::A_BYTES, STAGE_BYTES = Cfg::STAGE_BYTES, TMEM_COLS = Cfg::TMEM_COLS;
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  unsigned char* tiles = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  __shared__ __align__(8) uint64_t full_bar[STAGES], empty_bar[STAGES], acc_bar;
  __shared__ uint32_t s_tmem;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tok0 = blockIdx.x * TN, feat0 = blockIdx.y * DT_BM;
  const int ks = gridDim.z, rank = blockIdx.z;
  const int n_kb = (a.K + DT_BK - 1) / DT_BK;
  const int kb0 = (int)((long long)rank * n_kb / ks), nk = (int)((long long)(rank + 1) * n_kb / ks) - kb0;
  pdl_launch();

  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; s++) { mbar_init(&full_bar[s], 1); mbar_init(&empty_bar[s], 1); }
    mbar_init(&acc_bar, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(TMEM_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem_base = s_tmem;
  bool acc_ok = false;

  if (warp == 0 && lane == 0) {
    const int pre = nk < STAGES ? nk : STAGES;
    if (a.w_late) pdl_wait();
    auto load_w = [&](int i, int s) {
      unsigned char* st = tiles + (size_t)s * STAGE_BYTES;
      mbar_expect_tx(&full_bar[s], STAGE_BYTES);
      tma_load_2d(st, &tm_w0, (kb0 + i) * DT_BK, feat0, &full_bar[s]);
      if (NW == 2) tma_load_2d(st + A_BYTES, &tm_w1, (kb0 + i) * DT_BK, feat0, &full_bar[s]);
    };
    for (int i = 0; i < pre; i++) load_w(i, i);
    pdl_wait();  // the rows come from the previous kernel
    for (int i = 0; i < pre; i++)
      tma_load_2d(tiles + (size_t)i * STAGE_BYTES + NW * A_BYTES, &tm_x, (kb0 + i) * DT_BK, tok0, &full_bar[i]);
    for (int i = pre; i < nk; i++) {
      const int s = i % STAGES;
      if (!mbar_wait(&empty_bar[s], ((i / STAGES) - 1) & 1)) { atomicCAS(a.err, 0, 1); break; }
      load_w(i, s);
      tma_load_2d(tiles + (size_t)s * STAGE_BYTES + NW * A_BYTES, &tm_x, (kb0 + i) * DT_BK, tok0, &full_bar[s]);
    }
  } else if (warp == 1 && lane == 0) {
    // instruction descriptor: fp32 accumulator, bf16 x bf16, both operands K-major
    const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(TN >> 3) << 17) | ((uint32_t)(DT_BM >> 4) << 24);
    bool ok = true;
    pdl_wait();  // the poll budget starts once the predecessor is done
    for (int i = 0; i < nk; i++) {
      const int s = i % STAGES;
      if (!mbar_wait(&full_bar[s], (i / STAGES) & 1)) { atomicCAS(a.err, 0, 2); ok = false; break; }
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      unsigned char* st = tiles + (size_t)s * STAGE_BYTES;
      const uint64_t bdesc = umma_desc(st + NW * A_BYTES);
#pragma unroll
      for (int w = 0; w < NW; w++) {
        const uint64_t adesc = umma_desc(st + w * A_BYTES);
#pragma unroll
        for (int k = 0; k < DT_BK / 16; k++) umma_f16(tmem_base + w * TN, adesc + 2 * k, bdesc + 2 * k, idesc, (i > 0 || k > 0) ? 1u : 0u);
      }
      umma_commit(&empty_bar[s]);
    }
    if (ok) umma_commit(&acc_bar);
  } else if (warp >= 2) {
    pdl_wait();
    if (!GLU && a.out.act == JG_ACT_GELU_SIDE && rank == 0)  // the tile's rows of the token table, on their way while the product runs
      for (int t = (warp - 2) * 32 + lane; t < TN && tok0 + t < a.M; t += 128 * Cfg::EPW) {
        const bf16* p = dense_side_ptr<bf16>(a.out, a.out.tokens[tok0 + t], feat0);
        prefetch_l2(p);
        if (feat0 + 64 < a.N) prefetch_l2(p + 64);
      }
    acc_ok = mbar_wait(&acc_bar, 0);
    if (!acc_ok && lane == 0) atomicCAS(a.err, 0, 3);
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  }

  const int q = warp & 3, row = q * 32 + lane, part = (warp - 2) >> 2;
  constexpr int TN_PER = (TN / Cfg::EPW) >= 16 ? (TN / Cfg::EPW) : 16;
  constexpr int NC_PER = (NCOL / Cfg::EPW) >= 16 ? (NCOL / Cfg::EPW) : 16;
  const int tn_lo = part * TN_PER, tn_hi = min(TN, tn_lo + TN_PER);
  const int nc_lo = part * NC_PER, nc_hi = min(NCOL, nc_lo + NC_PER);
  const uint32_t t_lane = tmem_base + ((uint32_t)(q * 32) << 16);
  float* red = reinterpret_cast<float*>(tiles);  // rank 0: [ks-1][NCOL][128]
  if (ks > 1) {
    cluster_barrier();
    if (rank > 0 && warp >= 2 && acc_ok) {
      const uint32_t dst0 = map_to_rank(smem_u32(red + ((size_t)(rank - 1) * NCOL) * DT_BM + row), 0);
#pragma unroll 1
      for (int c0 = nc_lo; c0 < nc_hi; c0 += 16) {
        float r0[16];
        tmem_ld16(t_lane + c0, r0);
#pragma unroll
        for (int j = 0; j < 16; j++) st_cluster_f32(dst0 + (uint32_t)((c0 + j) * DT_BM * 4), r0[j]);
      }
    }
    cluster_barrier();
  }
  if (rank == 0 && warp >= 2 && acc_ok) {
    const int feat = feat0 + row;
    const float bias0 = (a.b0 && feat < a.N) ? a.b0[feat] : 0.f;
    const float bias1 = (NW == 2 && a.b1 && feat < a.N) ? a.b1[feat] : 0.f;
#pragma unroll 1
    for (int c0 = tn_lo; c0 < tn_hi; c0 += 16) {
      if (tok0 + c0 >= a.M) break;  // the same for all lanes of the warp
      float r0[16], r1[16];
      tmem_ld16(t_lane + c0, r0);
      if (NW == 2) tmem_ld16(t_lane + TN + c0, r1);
      for (int p = 1; p < ks; p++) {  // rank order
        const float* pr = red + ((size_t)(p - 1) * NCOL) * DT_BM + row;
#pragma unroll
        for (int j = 0; j < 16; j++) {
          r0[j] += pr[(size_t)(c0 + j) * DT_BM];
          if (NW == 2) r1[j] += pr[(size_t)(TN + c0 + j) * DT_BM];
        }
      }
      if (feat < a.N) {
        float side[16] = {};
        if (!GLU && a.out.act == JG_ACT_GELU_SIDE) {
#pragma unroll
          for (int j = 0; j < 16; j++) side[j] = dense_side<bf16>(a.out, min(tok0 + c0 + j, a.M - 1), feat);
        }
#pragma unroll
        for (int j = 0; j < 16; j++) {
          const int tok = tok0 + c0 + j;
          if (tok < a.M) {
            const size_t o = (size_t)tok * a.ldy + feat;
            if (GLU) a.y[o] = __float2bfloat16_rn(clamped_glu(r0[j] + bias0, r1[j] + bias1, a.limit));
            else {
              const float v = dense_act(a.out, feat, r0[j] + bias0, side[j]);
              if (feat >= a.out.split) a.out.y2[(size_t)tok * a.out.ld2 + feat - a.out.split] = v;
              else if (a.y32) a.y32[o] = v;
              else a.y[o] = __float2bfloat16_rn(v);
            }
          }
        }
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(TMEM_COLS) : "memory");
  }
}

template <int TN, bool GLU, bool HALF>
static int launch_dt(jg_dev* dev, const DenseCall& c, const DtArgs& a) {
  using Cfg = DtCfg<TN, GLU, HALF>;
  auto kern = dense_tc_kernel<TN, GLU, HALF>;
  static bool attr_set[8] = {};
  if (!attr_set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Cfg::SMEM));
    attr_set[dev->ordinal & 7] = true;
  }
  CUtensorMap tw0, tw1, tx;
  int rc = jg_tensor_map(&tw0, c.w[0], c.N, c.K, c.ldw, DT_BM, "weights", 2, true);
  if (rc) return rc;
  rc = jg_tensor_map(&tw1, c.w[GLU ? 1 : 0], c.N, c.K, c.ldw, DT_BM, "weights (second matrix)", 2, true);
  if (rc) return rc;
  rc = jg_tensor_map(&tx, c.x, c.M, c.K, c.ldx, TN, "activations", 2, true);
  if (rc) return rc;
  const int n_ft = (c.N + DT_BM - 1) / DT_BM, n_tt = (c.M + TN - 1) / TN, tiles = n_ft * n_tt, n_kb = (c.K + DT_BK - 1) / DT_BK;
  int ks = 1;
  if (c.M > 128) {  // the split with the smallest waves x (k-blocks at the tensor peak + fixed cost) estimate, as in gemm_tc.cu
    float best = 0.f;
    for (int s = 1; s <= Cfg::MAX_KS && s <= 8 && n_kb / s >= 8; s++) {
      const int slots = dev->sm_count * (HALF ? 2 : 1), waves = (tiles * s + slots - 1) / slots;
      const float t = (float)waves * ((float)(n_kb / s) * 0.28f + 18.f);
      if (s == 1 || t < best) { best = t; ks = s; }
    }
  } else {
    while (ks < (HALF && tiles > 8 ? 4 : 8) && ks < Cfg::MAX_KS && tiles * ks * 3 < dev->sm_count * 2 * (HALF ? 2 : 1) && n_kb / (ks + 1) >= 8) ks++;
  }
  dev->tc_pending = true;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(n_tt, n_ft, ks);
  cfg.blockDim = dim3(Cfg::THREADS);
  cfg.dynamicSmemBytes = Cfg::SMEM;
  cfg.stream = dev->stream;
  cudaLaunchAttribute attr[2];
  int na = 0;
  if (ks > 1) {
    attr[na].id = cudaLaunchAttributeClusterDimension;
    attr[na].val.clusterDim.x = 1;
    attr[na].val.clusterDim.y = 1;
    attr[na].val.clusterDim.z = ks;
    na++;
  }
  if (dev->pdl) {
    attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[na].val.programmaticStreamSerializationAllowed = 1;
    na++;
  }
  cfg.attrs = attr;
  cfg.numAttrs = na;
  cudaError_t e = cudaLaunchKernelEx(&cfg, kern, tw0, tw1, tx, a);
  if (e != cudaSuccess) return jg_cuda_fail(e, "dense_tc", __FILE__, __LINE__);
  return jg_after_launch(dev, "dense_tc");
}

int jg_dense_tc(jg_dev* dev, const DenseCall& c) {
  JG_REQUIRE(((uintptr_t)c.x % 16) == 0 && c.ldx % 8 == 0 && c.ldw % 8 == 0, "dense: operands must be 16-byte aligned with row strides of a multiple of 8");
  if (dev->err_word == nullptr) {
    JG_REQUIRE(!dev->capturing, "first tensor-core projection on a device must not be inside a graph capture");
    JG_CUDA(cudaMalloc(&dev->err_word, sizeof(int)));
    JG_CUDA(cudaMemsetAsync(dev->err_word, 0, sizeof(int), dev->stream));
  }
  DtArgs a = {};
  if (c.out_f32) a.y32 = (float*)c.y;
  else a.y = (bf16*)c.y;
  a.b0 = c.bias[0]; a.b1 = c.bias[1]; a.err = dev->err_word; a.M = c.M; a.N = c.N; a.K = c.K; a.ldy = c.ldy; a.limit = c.limit; a.out = c.out;
  a.w_late = jg_is_fresh(dev, c.w[0]) || jg_is_fresh(dev, c.w[1]);
  if (c.epilogue == JG_DENSE_GLU) {
    if (c.M <= 16) return launch_dt<16, true, false>(dev, c, a);
    if (c.M <= 32) return launch_dt<32, true, false>(dev, c, a);
    if (c.M <= 64) return launch_dt<64, true, false>(dev, c, a);
    if (c.M <= 128) return launch_dt<128, true, false>(dev, c, a);
    return launch_dt<256, true, false>(dev, c, a);
  }
  if (c.M <= 16) return launch_dt<16, false, true>(dev, c, a);
  if (c.M <= 32) return launch_dt<32, false, true>(dev, c, a);
  // few features: narrow tiles, two CTAs per SM and a deep split, so that there are CTAs enough; a short K: the same by tiles alone
  if (c.N <= 512) return launch_dt<32, false, true>(dev, c, a);
  if (c.M <= 64) return launch_dt<64, false, false>(dev, c, a);
  const bool few = c.K <= 512 && (c.N + DT_BM - 1) / DT_BM * ((c.M + 255) / 256) < dev->sm_count;
  if (c.M <= 128 || few) return launch_dt<128, false, false>(dev, c, a);
  return launch_dt<256, false, false>(dev, c, a);
}
