// Matmul over bfloat16 weights for prompts and batches of 16 and more of the block models:
//   Y[t][row] = act(sum_k W[row][k] * X[t][k])      (W and X bfloat16, FP32 accumulation)
//
// dense_gemm_kernel: 5th-generation tensor cores, one persistent CTA per SM. Weight rows are the MMA's M side (128 per
// tile), tokens its N side (32 to 256 per tile). A producer lane moves both operands' 64-element K slices with TMA
// (cp.async.bulk.tensor.2d, 128-byte swizzle; rows, tokens and elements beyond the matrices read as zero, so every
// size is served), an MMA lane issues tcgen05.mma into one of two accumulators in tensor memory, and eight warps read the
// other one back (tcgen05.ld) and apply the segment's activation: a tile's epilogue runs under the next tile's products.
// Token tiles of the same weight rows follow one another, so a weight row comes from HBM once. Launches with few tiles
// (small batches) split K: partial tiles go to a workspace and the last CTA of a tile adds them in order.
// Segments (the projections of one input) share a launch; each has its own weights, activation rows and output.
//
// sgemm_kernel: the same product in plain FP32 arithmetic (FFMA on FP32 activations; the bfloat16 weights are exact in
// FP32), for engines that run in 32-bit.
#pragma once
#include "dense_gemv.cuh"
#include "gemm_tc.cuh"

namespace b200 {

constexpr int DGM_EPI_WARPS = 8;
constexpr int DGM_THREADS = 32 * DGM_EPI_WARPS + 64;  // + the TMA warp and the MMA warp
constexpr int DGM_MAX_STAGES = 8;
constexpr int DGM_SMEM = 216 * 1024;

struct DgmSeg {
  const __nv_bfloat16* w;  // [rows][pad8(K)]
  const void* x;           // [T][x_ld] bfloat16 (sgemm: FP32)
  int x_ld;
  int rows;                // matrix rows (gated products: interleaved gate and up rows)
  int outs;                // outputs (= rows, or the inner size of the gated product)
  int act;
  void* y;                 // [T][y_stride], FP32 or bfloat16
  int y_stride;
  int y_bf16;
  const float* bias;       // [rows], or nullptr
  float arg;               // cap of ACT_SOFTCAP
};

struct DgmParams {
  DgmSeg seg[DGV_MAX_SEGS];
  int nseg, K, T;
  int NT, stages, acc_cols;    // token tile, ring depth, tensor-memory columns per accumulator
  int tiles_m, tiles_n;        // 128-row tiles over all segments, token tiles
  int ksplit, ksteps;          // K splits and 64-element steps per split
  float* ws;                   // split K: partial tiles [ksplit][tile][NT][128]
  int* tickets;                // split K: one per tile, zero between launches
  int* error_flag;
};

struct alignas(64) DgmMaps {
  CUtensorMap w[DGV_MAX_SEGS], x[DGV_MAX_SEGS];
};

struct DgmShared {
  unsigned long long full[DGM_MAX_STAGES], empty[DGM_MAX_STAGES], acc_full[2], acc_empty[2];
  uint32_t tmem_base;
  int abort_flag, issued;  // issued: K slices whose copies have been requested
  int last;
};

// kind::f16 with bfloat16 operands: D = F32, A and B = BF16 and K-major
__host__ __device__ __forceinline__ uint32_t dgm_idesc(int n) { return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(TC_M >> 4) << 24); }

__device__ __forceinline__ bool dgm_wait(const DgmParams& p, DgmShared* sh, void* bar, uint32_t parity) {
  if (*(volatile int*)&sh->abort_flag) return false;
  if (mbar_wait(bar, parity)) return true;
  *(volatile int*)&sh->abort_flag = 1;
  if (p.error_flag) *reinterpret_cast<volatile int*>(p.error_flag) = 1;
  return false;
}

// this warp's 32 TMEM lanes, 16 consecutive columns
__device__ __forceinline__ void tc_ld16(uint32_t taddr, float (&v)[16]) {
  uint32_t r[16];
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
                 "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
               : "r"(taddr));
  asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
  for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]);
}

__device__ __forceinline__ void dgm_put(float* y, float v) { *y = v; }
__device__ __forceinline__ void dgm_put(__nv_bfloat16* y, float v) { *y = __float2bfloat16(v); }

// Sixteen columns (tokens t0 ..) of this lane's row: activation and store. ACT is a compile-time copy of sg.act.
template <int ACT, typename Y>
__device__ __forceinline__ void dgm_store16(const DgmSeg& sg, int row, int t0, int T, float bias, const float (&v)[16]) {
  if (act_is_glu(ACT)) {
    const int o = (row >> 4) * 8 + (row & 7);
    const bool mine = !(row & 8) && o < sg.outs;
    Y* y = static_cast<Y*>(sg.y) + (size_t)t0 * sg.y_stride + o;
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      const float up = __shfl_sync(0xffffffffu, v[j], ((threadIdx.x & 31) & 23) + 8);
      if (mine && t0 + j < T) dgm_put(y, glu_act(ACT, v[j], up));
      y += sg.y_stride;
    }
  } else if (row < sg.rows) {
    Y* y = static_cast<Y*>(sg.y) + (size_t)t0 * sg.y_stride + row;
    const int n = min(16, T - t0);
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      if (j < n) dgm_put(y, dense_act(ACT, v[j] + bias, sg.arg));
      y += sg.y_stride;
    }
  }
}
template <typename Y>
__device__ __forceinline__ void dgm_store16(const DgmSeg& sg, int row, int t0, int T, float bias, const float (&v)[16]) {
  switch (sg.act) {
    case ACT_SIGMOID: dgm_store16<ACT_SIGMOID, Y>(sg, row, t0, T, bias, v); break;
    case ACT_SILU: dgm_store16<ACT_SILU, Y>(sg, row, t0, T, bias, v); break;
    case ACT_TANH: dgm_store16<ACT_TANH, Y>(sg, row, t0, T, bias, v); break;
    case ACT_DECAY: dgm_store16<ACT_DECAY, Y>(sg, row, t0, T, bias, v); break;
    case ACT_GELU: dgm_store16<ACT_GELU, Y>(sg, row, t0, T, bias, v); break;
    case ACT_SOFTCAP: dgm_store16<ACT_SOFTCAP, Y>(sg, row, t0, T, bias, v); break;
    case ACT_SILU_GLU: dgm_store16<ACT_SILU_GLU, Y>(sg, row, t0, T, bias, v); break;
    case ACT_RELU_GLU: dgm_store16<ACT_RELU_GLU, Y>(sg, row, t0, T, bias, v); break;
    default: dgm_store16<ACT_NONE, Y>(sg, row, t0, T, bias, v);
  }
}

__host__ __device__ __forceinline__ size_t dgm_stage_bytes(int NT) { return (size_t)TC_M * 128 + (size_t)NT * 128; }

// One unit of work: a tile of 128 rows x NT tokens over a range of K.
struct DgmUnit {
  int seg, row0, t0, tile, k0, steps;
};
__device__ __forceinline__ DgmUnit dgm_unit(const DgmParams& p, int u) {
  DgmUnit r;
  const int n = u % p.tiles_n, rest = u / p.tiles_n, kz = rest % p.ksplit;
  int m = rest / p.ksplit;
  r.tile = m * p.tiles_n + n;
  r.seg = 0;
  while (r.seg + 1 < p.nseg && m >= (p.seg[r.seg].rows + TC_M - 1) / TC_M) { m -= (p.seg[r.seg].rows + TC_M - 1) / TC_M; ++r.seg; }
  r.row0 = m * TC_M;
  r.t0 = n * p.NT;
  r.k0 = kz * p.ksteps;
  r.steps = min(p.ksteps, (p.K + TC_KC - 1) / TC_KC - r.k0);
  return r;
}

// grid = min(units, SMs)
__global__ void __launch_bounds__(DGM_THREADS, 1) dense_gemm_kernel(const DgmParams p, const __grid_constant__ DgmMaps maps) {
  extern __shared__ uint8_t dgm_smem_raw[];
  __shared__ DgmShared sh;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  uint8_t* smem = reinterpret_cast<uint8_t*>(((uintptr_t)dgm_smem_raw + 1023) & ~(uintptr_t)1023);
  const uint32_t stage_bytes = (uint32_t)dgm_stage_bytes(p.NT);
  const int units = p.tiles_m * p.tiles_n * p.ksplit;
  if (tid == 0) {
    for (int i = 0; i < DGM_MAX_STAGES; ++i) { mbar_init(&sh.full[i], 1); mbar_init(&sh.empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&sh.acc_full[i], 1); mbar_init(&sh.acc_empty[i], DGM_EPI_WARPS); }
    sh.abort_flag = 0;
    sh.issued = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) tc_alloc(&sh.tmem_base, 2 * p.acc_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sh.tmem_base;

  if (warp == DGM_EPI_WARPS) {
    // ---- producer lane ----
    if (lane == 0) {
      int s = 0, st = 0;
      uint32_t ph = 1;  // a fresh ring's slots count as empty
      bool ok = true;
      for (int u = blockIdx.x; u < units && ok; u += gridDim.x) {
        const DgmUnit w = dgm_unit(p, u);
        for (int k = 0; k < w.steps; ++k) {
          if (s >= p.stages && !(ok = dgm_wait(p, &sh, &sh.empty[st], ph))) break;
          uint8_t* a = smem + (size_t)st * stage_bytes;
          mbar_expect_tx(&sh.full[st], stage_bytes);
          tc_tma_load_2d(a, &maps.w[w.seg], (w.k0 + k) * TC_KC, w.row0, &sh.full[st]);
          tc_tma_load_2d(a + TC_M * 128, &maps.x[w.seg], (w.k0 + k) * TC_KC, w.t0, &sh.full[st]);
          sh.issued = ++s;
          if (++st == p.stages) { st = 0; ph ^= 1u; }
        }
      }
    }
    __syncwarp();
  } else if (warp == DGM_EPI_WARPS + 1) {
    // ---- MMA lane ----
    if (lane == 0) {
      const uint32_t idesc = dgm_idesc(p.NT);
      int st = 0, n = 0;
      uint32_t ph = 0;
      bool ok = true;
      for (int u = blockIdx.x; u < units && ok; u += gridDim.x, ++n) {
        const DgmUnit w = dgm_unit(p, u);
        const int buf = n & 1;
        if (n >= 2 && !(ok = dgm_wait(p, &sh, &sh.acc_empty[buf], (uint32_t)((n / 2 - 1) & 1)))) break;
        tc_fence_after();
        const uint32_t d = tmem + (uint32_t)(buf * p.acc_cols);
        for (int k = 0; k < w.steps; ++k) {
          if (!(ok = dgm_wait(p, &sh, &sh.full[st], ph))) break;
          tc_fence_after();
          const uint32_t a = smem_u32(smem + (size_t)st * stage_bytes);
          const uint64_t ad = tc_smem_desc(a), bd = tc_smem_desc(a + TC_M * 128);
#pragma unroll
          for (int k4 = 0; k4 < 4; ++k4) tc_mma_f16(d, ad + 2 * k4, bd + 2 * k4, idesc, (k | k4) ? 1u : 0u);
          tc_commit(&sh.empty[st]);
          if (++st == p.stages) { st = 0; ph ^= 1u; }
        }
        if (ok) tc_commit(&sh.acc_full[buf]);
      }
    }
    __syncwarp();
  } else {
    // ---- epilogue warps: lanes 32 (w & 3) .. of the accumulator = weight rows, the two groups of four split the tokens ----
    const int r = 32 * (warp & 3) + lane, c_begin = (warp >> 2) * (p.NT / 2), c_end = c_begin + p.NT / 2;
    auto store = [&](const DgmSeg& sg, int row, int t0, float bias, const float (&v)[16]) {
      if (sg.y_bf16) dgm_store16<__nv_bfloat16>(sg, row, t0, p.T, bias, v);
      else dgm_store16<float>(sg, row, t0, p.T, bias, v);
    };
    int n = 0;
    for (int u = blockIdx.x; u < units; u += gridDim.x, ++n) {
      const DgmUnit w = dgm_unit(p, u);
      const int buf = n & 1;
      const uint32_t parity = (uint32_t)((n / 2) & 1);
      if (p.ksplit > 1) {  // one decision for all epilogue warps: they meet on barriers below
        if (tid == 0) sh.last = dgm_wait(p, &sh, &sh.acc_full[buf], parity);
        asm volatile("bar.sync 1, %0;" ::"n"(32 * DGM_EPI_WARPS) : "memory");
        const bool go = sh.last != 0;
        asm volatile("bar.sync 1, %0;" ::"n"(32 * DGM_EPI_WARPS) : "memory");
        if (!go) break;
        mbar_wait(&sh.acc_full[buf], parity);  // complete already: orders this thread's reads
        __syncwarp();
      } else if (!__shfl_sync(0xffffffffu, (int)(lane == 0 ? dgm_wait(p, &sh, &sh.acc_full[buf], parity) : 0), 0)) {
        break;  // one decision per warp: the loads below need all its lanes
      }
      tc_fence_after();
      const DgmSeg& sg = p.seg[w.seg];
      const int row = w.row0 + r;
      const float bias = sg.bias && row < sg.rows ? sg.bias[row] : 0.f;
      const uint32_t base = tmem + ((uint32_t)(32 * (warp & 3)) << 16) + (uint32_t)(buf * p.acc_cols);
      float* part = p.ws + ((size_t)((w.k0 / p.ksteps) * p.tiles_m * p.tiles_n + w.tile) * p.NT) * TC_M + r;
      for (int c = c_begin; c < c_end && w.t0 + c < p.T; c += 16) {
        float v[16];
        tc_ld16(base + (uint32_t)c, v);
        if (p.ksplit > 1) {
#pragma unroll
          for (int j = 0; j < 16; ++j) part[(size_t)(c + j) * TC_M] = v[j];
        } else {
          store(sg, row, w.t0 + c, bias, v);
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.acc_empty[buf]);
      if (p.ksplit > 1) {
        __threadfence();
        asm volatile("bar.sync 1, %0;" ::"n"(32 * DGM_EPI_WARPS) : "memory");
        if (tid == 0) {
          sh.last = atomicAdd(&p.tickets[w.tile], 1) == p.ksplit - 1;
          if (sh.last) p.tickets[w.tile] = 0;
        }
        asm volatile("bar.sync 1, %0;" ::"n"(32 * DGM_EPI_WARPS) : "memory");
        if (sh.last) {
          __threadfence();
          const size_t step = (size_t)p.tiles_m * p.tiles_n * p.NT * TC_M;
          const float* sum = p.ws + (size_t)w.tile * p.NT * TC_M + r;
          for (int c = c_begin; c < c_end && w.t0 + c < p.T; c += 16) {
            float v[16];
#pragma unroll
            for (int j = 0; j < 16; ++j) v[j] = 0.f;
            for (int z = 0; z < p.ksplit; ++z)
#pragma unroll
              for (int j = 0; j < 16; ++j) v[j] += __ldcg(sum + z * step + (size_t)(c + j) * TC_M);
            store(sg, row, w.t0 + c, bias, v);
          }
        }
        asm volatile("bar.sync 1, %0;" ::"n"(32 * DGM_EPI_WARPS) : "memory");  // sh.last is read before the next unit writes it
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  // The MMA lane waits for every copy; only after a give-up may some still be in flight, and the block outlives them.
  if (sh.abort_flag && tid == 0)
    for (int s = max(0, sh.issued - p.stages); s < sh.issued; ++s) mbar_wait(&sh.full[s % p.stages], (uint32_t)((s / p.stages) & 1));
  if (warp == 0) tc_dealloc(tmem, 2 * p.acc_cols);
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
  const bool glu = act_is_glu(sg.act);
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
        if (glu && half == 0) { kept[i][j] = acc[i][j]; continue; }
        if (row >= sg.outs || t >= p.T) continue;
        const float v = glu ? glu_act(sg.act, kept[i][j], acc[i][j]) : dense_act(sg.act, acc[i][j] + (sg.bias ? sg.bias[row] : 0.f), sg.arg);
        if (sg.y_bf16) static_cast<__nv_bfloat16*>(sg.y)[(size_t)t * sg.y_stride + row] = __float2bfloat16(v);
        else static_cast<float*>(sg.y)[(size_t)t * sg.y_stride + row] = v;
      }
  }
}

}  // namespace b200
