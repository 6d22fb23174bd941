// Matmul over bfloat16 weights for prompts and batches of 16 and more of the block models:
//   Y[t][row] = act(sum_k W[row][k] * X[t][k])      (W and X bfloat16, FP32 accumulation)
//
// dense_gemm_kernel: 5th-generation tensor cores. Weight rows are the MMA's M side (128 per CTA tile), tokens its N
// side (32 to 256 per tile). A producer lane moves both operands' 64-element K slices with TMA
// (cp.async.bulk.tensor.2d, 128-byte swizzle; rows, tokens and elements beyond the matrices read as zero, so every
// size is served), an MMA lane issues tcgen05.mma into a 128-lane x NT-column FP32 tile in tensor memory, four warps
// read it back (tcgen05.ld) and apply the segment's activation. Two CTAs share an SM (at most 256 tensor-memory columns
// each), so one tile's epilogue overlaps the other's products. Segments (the projections of one input) share a launch;
// each has its own weights, activation rows and output.
//
// sgemm_kernel: the same product in plain FP32 arithmetic (FFMA on FP32 activations; the bfloat16 weights are exact in
// FP32), for engines that run in 32-bit.
#pragma once
#include "dense_gemv.cuh"
#include "gemm_tc.cuh"

namespace b200 {

constexpr int DGM_THREADS = 192;  // four epilogue warps, the TMA warp, the MMA warp
constexpr int DGM_MAX_STAGES = 8;
constexpr int DGM_SMEM_PER_CTA = 110 * 1024;  // two CTAs per SM

struct DgmSeg {
  const __nv_bfloat16* w;  // [rows][pad8(K)]
  const void* x;           // [T][x_ld] bfloat16 (sgemm: FP32)
  int x_ld;
  int rows;                // matrix rows (ACT_RELU_GLU: interleaved gate and up rows)
  int outs;                // outputs (= rows, or the inner size of the gated product)
  int act;
  void* y;                 // [T][y_stride], FP32 or bfloat16
  int y_stride;
  int y_bf16;
  const float* aux;        // per-row bias of ACT_DECAY
};

struct DgmParams {
  DgmSeg seg[DGV_MAX_SEGS];
  int nseg, K, T;
  int NT, stages, tmem_cols;
  int* error_flag;
};

struct alignas(64) DgmMaps {
  CUtensorMap w[DGV_MAX_SEGS], x[DGV_MAX_SEGS];
};

struct DgmShared {
  unsigned long long full[DGM_MAX_STAGES], empty[DGM_MAX_STAGES], done;
  uint32_t tmem_base;
  int abort_flag, issued;  // steps whose copies have been issued
};

// kind::f16 with bfloat16 operands: D = F32, A and B = BF16 and K-major
__host__ __device__ __forceinline__ uint32_t dgm_idesc(int n) { return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(TC_M >> 4) << 24); }

__device__ __forceinline__ void dgm_fail(const DgmParams& p, DgmShared* sh) {
  *(volatile int*)&sh->abort_flag = 1;
  if (p.error_flag) *reinterpret_cast<volatile int*>(p.error_flag) = 1;
}

__device__ __forceinline__ void dgm_store(const DgmSeg& sg, int t, int row, float v) {
  if (sg.y_bf16) static_cast<__nv_bfloat16*>(sg.y)[(size_t)t * sg.y_stride + row] = __float2bfloat16(v);
  else static_cast<float*>(sg.y)[(size_t)t * sg.y_stride + row] = v;
}

__host__ __device__ __forceinline__ size_t dgm_stage_bytes(int NT) { return (size_t)TC_M * 128 + (size_t)NT * 128; }

// grid = (128-row tiles over all segments, token tiles)
__global__ void __launch_bounds__(DGM_THREADS, 2) dense_gemm_kernel(const DgmParams p, const __grid_constant__ DgmMaps maps) {
  extern __shared__ uint8_t dgm_smem_raw[];
  __shared__ DgmShared sh;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  uint8_t* smem = reinterpret_cast<uint8_t*>(((uintptr_t)dgm_smem_raw + 1023) & ~(uintptr_t)1023);
  const uint32_t stage_bytes = (uint32_t)dgm_stage_bytes(p.NT);
  int seg = 0, mt = blockIdx.x;
  while (seg + 1 < p.nseg && mt >= (p.seg[seg].rows + TC_M - 1) / TC_M) { mt -= (p.seg[seg].rows + TC_M - 1) / TC_M; ++seg; }
  const DgmSeg& sg = p.seg[seg];
  const int row0 = mt * TC_M, t0 = blockIdx.y * p.NT;
  const int nsteps = (p.K + TC_KC - 1) / TC_KC;
  if (tid == 0) {
    for (int i = 0; i < DGM_MAX_STAGES; ++i) { mbar_init(&sh.full[i], 1); mbar_init(&sh.empty[i], 1); }
    mbar_init(&sh.done, 1);
    sh.abort_flag = 0;
    sh.issued = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) tc_alloc(&sh.tmem_base, p.tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_d = sh.tmem_base;

  if (warp == 4) {
    if (lane == 0) {
      for (int s = 0; s < nsteps; ++s) {
        const int st = s % p.stages;
        if (s >= p.stages && !mbar_wait(&sh.empty[st], (uint32_t)((s / p.stages - 1) & 1))) { dgm_fail(p, &sh); break; }
        uint8_t* a = smem + (size_t)st * stage_bytes;
        mbar_expect_tx(&sh.full[st], stage_bytes);
        tc_tma_load_2d(a, &maps.w[seg], s * TC_KC, row0, &sh.full[st]);
        tc_tma_load_2d(a + TC_M * 128, &maps.x[seg], s * TC_KC, t0, &sh.full[st]);
        sh.issued = s + 1;
      }
    }
    __syncwarp();
  } else if (warp == 5) {
    if (lane == 0) {
      const uint32_t idesc = dgm_idesc(p.NT);
      bool ok = true;
      for (int s = 0; s < nsteps && ok; ++s) {
        const int st = s % p.stages;
        ok = mbar_wait(&sh.full[st], (uint32_t)((s / p.stages) & 1));
        if (!ok) break;
        tc_fence_after();
        const uint32_t a = smem_u32(smem + (size_t)st * stage_bytes);
        const uint64_t ad = tc_smem_desc(a), bd = tc_smem_desc(a + TC_M * 128);
#pragma unroll
        for (int k4 = 0; k4 < 4; ++k4) tc_mma_f16(tmem_d, ad + 2 * k4, bd + 2 * k4, idesc, (s | k4) ? 1u : 0u);
        tc_commit(&sh.empty[st]);
      }
      if (!ok) dgm_fail(p, &sh);
      tc_commit(&sh.done);
    }
    __syncwarp();
  } else {
    if (!mbar_wait(&sh.done, 0u)) dgm_fail(p, &sh);
    __syncwarp();
    tc_fence_after();
    if (!*(volatile int*)&sh.abort_flag) {
      const int row = row0 + 32 * warp + lane;
      const float aux = sg.aux && row < sg.rows ? sg.aux[row] : 0.f;
      for (int c0 = 0; c0 < p.NT && t0 + c0 < p.T; c0 += 8) {
        float v[8];
        tc_ld8(tmem_d + ((uint32_t)(32 * warp) << 16) + (uint32_t)c0, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const int t = t0 + c0 + j;
          if (sg.act == ACT_RELU_GLU) {
            const float up = __shfl_sync(0xffffffffu, v[j], (lane & 23) + 8);
            const int o = (row >> 4) * 8 + (row & 7);
            if (!(row & 8) && o < sg.outs && t < p.T) dgm_store(sg, t, o, fmaxf(v[j], 0.f) * up);
          } else if (row < sg.rows && t < p.T) {
            dgm_store(sg, t, row, dense_act(sg.act, v[j], aux));
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  // The MMA lane waits for every copy; only after a give-up may some still be in flight, and the block outlives them.
  if (sh.abort_flag && tid == 0)
    for (int s = max(0, sh.issued - p.stages); s < sh.issued; ++s) mbar_wait(&sh.full[s % p.stages], (uint32_t)((s / p.stages) & 1));
  if (warp == 0) tc_dealloc(tmem_d, p.tmem_cols);
}

// 64 rows x 64 tokens per block of 256 threads, 4 x 4 outputs per thread, K in steps of 16. grid = (row tiles over all
// segments, token tiles). FP32 activations with a stride of pad8(K) or more.
__global__ void __launch_bounds__(256) sgemm_kernel(const DgmParams p) {
  __shared__ float ws[16][64 + 4], xs[16][64 + 4];
  const int tid = threadIdx.x;
  int seg = 0, mt = blockIdx.x;
  auto tiles = [&](int s) { return (p.seg[s].outs + 63) / 64; };
  while (seg + 1 < p.nseg && mt >= tiles(seg)) { mt -= tiles(seg); ++seg; }
  const DgmSeg& sg = p.seg[seg];
  const bool glu = sg.act == ACT_RELU_GLU;
  const int ld = pad8(p.K), r0 = mt * 64, t0 = blockIdx.y * 64;
  const int tr = tid & 15, tt = tid >> 4;
  float kept[4][4];  // the gated product keeps its gate half while the up half is computed
  for (int half = 0; half < (glu ? 2 : 1); ++half) {
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < p.K; k0 += 16) {
      for (int i = tid; i < 64 * 16; i += 256) {
        const int r = i >> 4, k = k0 + (i & 15);
        float w = 0.f, x = 0.f;
        if (k < p.K && r0 + r < sg.outs) w = __bfloat162float(sg.w[(size_t)(glu ? glu_row(r0 + r, half) : r0 + r) * ld + k]);
        if (k < p.K && t0 + r < p.T) x = static_cast<const float*>(sg.x)[(size_t)(t0 + r) * sg.x_ld + k];
        ws[i & 15][r] = w;
        xs[i & 15][r] = x;
      }
      __syncthreads();
#pragma unroll
      for (int k = 0; k < 16; ++k) {
        const float4 w = *reinterpret_cast<const float4*>(&ws[k][4 * tr]), x = *reinterpret_cast<const float4*>(&xs[k][4 * tt]);
        const float wv[4] = {w.x, w.y, w.z, w.w}, xv[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(wv[i], xv[j], acc[i][j]);
      }
      __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int row = r0 + 4 * tr + i, t = t0 + 4 * tt + j;
        if (glu && half == 0) { kept[i][j] = fmaxf(acc[i][j], 0.f); continue; }
        if (row >= sg.outs || t >= p.T) continue;
        dgm_store(sg, t, row, glu ? kept[i][j] * acc[i][j] : dense_act(sg.act, acc[i][j], sg.aux ? sg.aux[row] : 0.f));
      }
  }
}

}  // namespace b200
