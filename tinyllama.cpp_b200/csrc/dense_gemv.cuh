// Matvec over bfloat16 weights for decode batches of the block models, with the layer's row work fused in.
//
// Prologue (every CTA repeats it for the vectors it needs; one CTA stores what the rest of the step reads):
//   1. the pending sublayer output is added to the residual stream, normalised if it has a norm of its own:
//      x <- x + rms(add) * add_w, or x <- x + add; a looped stretch may then add its embedding rows once more;
//   2. the stream is normalised for this launch: h = rms(x) * norm_w;
//   3. token-shift launches mix h with the previous token's h, with one mix per segment: h + (h' - h) * mu_seg.
// Each step is optional. Activations stay in FP32 in shared memory, weights are read once from HBM as 16-byte pieces
// straight into registers, products and sums are FP32. Epilogue per segment: bias and activation, or the gated product
// act(gate) * up whose two rows one warp owns, or the logits with argmax partials and repetition penalty.
//
// A warp owns two rows; K is walked in pieces of 8 elements per lane, four pieces of both rows in flight. The pieces
// of a warp's first task are requested before the launch waits for the previous kernel (programmatic dependent launch):
// weights depend on nothing. Up to NB activation vectors share one pass over the weights; grid.y covers larger batches.
// Rows may have any length: they are stored with a stride of a multiple of 8 elements, zero-filled.
#pragma once
#include <cuda_bf16.h>

#include "gemv.cuh"

namespace b200 {

enum : int { ACT_NONE = 0, ACT_SIGMOID, ACT_SILU, ACT_TANH, ACT_DECAY, ACT_GELU, ACT_SOFTCAP, ACT_RELU_GLU, ACT_SILU_GLU };

__host__ __device__ __forceinline__ bool act_is_glu(int act) { return act >= ACT_RELU_GLU; }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
// 2^x and 1 / x of the special-function unit: FP32 to within two units in the last place, tiny results become zero
__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_fast(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// z * sigmoid(w): SiLU with w = z; GELU (tanh form, 0.5 z (1 + tanh(v)) = z sigmoid(2v)) with w = 2v
__device__ __forceinline__ float swish_f(float z, float w) { return z * rcp_fast(1.0f + ex2_fast(-1.4426950408889634f * w)); }
__device__ __forceinline__ float gelu_tanh_f(float z) { return swish_f(z, 1.5957691216057308f * (z + 0.044715f * z * z * z)); }
__device__ __forceinline__ float softcap_f(float z, float cap) { return cap * tanhf(z / cap); }
// v: the row's product with its bias added; arg: the cap of ACT_SOFTCAP
__device__ __forceinline__ float dense_act(int act, float v, float arg) {
  switch (act) {
    case ACT_SIGMOID: return sigmoid_f(v);
    case ACT_SILU: return swish_f(v, v);
    case ACT_TANH: return tanhf(v);
    case ACT_DECAY: return expf(-expf(v));
    case ACT_GELU: return gelu_tanh_f(v);
    case ACT_SOFTCAP: return softcap_f(v, arg);
    default: return v;
  }
}
__device__ __forceinline__ float glu_act(int act, float gate, float up) { return (act == ACT_SILU_GLU ? swish_f(gate, gate) : fmaxf(gate, 0.f)) * up; }

__host__ __device__ __forceinline__ int pad8(int n) { return (n + 7) & ~7; }
// Gate and up rows of a gated feed-forward share one matrix: eight gate rows, then the same eight up rows.
__host__ __device__ __forceinline__ int64_t glu_row(int64_t r, int half) { return ((r >> 3) << 4) + (r & 7) + 8 * half; }

constexpr int DGV_MAX_SEGS = 5;
constexpr int DGV_WARPS = 16, DGV_THREADS = 32 * DGV_WARPS;
constexpr int DGV_U = 4;  // 16-byte pieces of each row in flight per lane

struct DgvSeg {
  const __nv_bfloat16* w;  // [rows][ld] (gated products: gate / up rows interleaved, rows = outputs)
  int rows, act;
  float* y;                // [batch][y_stride]
  int y_stride;
  const float* mu;         // token shift: this segment's mix, or nullptr
  const float* bias;       // [rows], or nullptr
  float arg;               // cap of ACT_SOFTCAP
};

struct DgvParams {
  DgvSeg seg[DGV_MAX_SEGS];
  int nseg, K, batch;
  const float* x;          // [batch][x_stride]
  int x_stride;
  const float* add;        // pending sublayer output [batch][x_stride], or nullptr
  const float* add_w;      // its norm, or nullptr: added as it is
  const float* add2;       // further rows added to the stream [batch][x_stride] (only with add), or nullptr
  float* x_out;            // the new residual stream [batch][x_stride] (another buffer than x)
  const float* norm_w;     // nullptr: the input is used as it is
  float eps;
  // token shift: the previous token's h of every slot, two copies selected by the position's parity
  float* shift;            // [slot][2][shift_stride]
  int shift_stride;
  const int* positions;
  const int* slots;
  int ctas_per_seg;        // token shift: every segment has CTAs of its own (grid.x = nseg * ctas_per_seg); 0: CTAs share the segments
  // logits: argmax partials [batch][gridDim.x] and the repetition penalty (see GemvParams)
  float* amax_val;
  int* amax_idx;
  const uint8_t* pen_counts;
  int pen_stride;
  const float* pen_value;
};

__host__ __device__ __forceinline__ size_t dgv_smem_bytes(int K, int nb) { return (size_t)nb * pad8(K) * 4; }

// four consecutive elements, those at or beyond n read as zero
__device__ __forceinline__ float4 ld4_masked(const float* p, int i, int n) {
  float4 v = *reinterpret_cast<const float4*>(p + i);
  if (i + 3 >= n) {
    if (i >= n) v.x = 0.f;
    if (i + 1 >= n) v.y = 0.f;
    if (i + 2 >= n) v.z = 0.f;
    v.w = 0.f;
  }
  return v;
}

__device__ __forceinline__ float bf_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf_hi(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }

// Sums NB values over the block; every thread gets the totals.
template <int NB, int WARPS>
__device__ __forceinline__ void block_sums(float (&v)[NB], float* scratch /* [WARPS * NB] */) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
  for (int n = 0; n < NB; ++n) {
    v[n] = warp_sum(v[n]);
    if (lane == 0) scratch[warp * NB + n] = v[n];
  }
  __syncthreads();
#pragma unroll
  for (int n = 0; n < NB; ++n) {
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) t += scratch[w * NB + n];
    v[n] = t;
  }
  __syncthreads();
}

template <int NB>
__global__ void __launch_bounds__(DGV_THREADS, NB <= 2 ? 2 : 1) dense_gemv_kernel(const DgvParams p) {
  extern __shared__ __align__(16) float dgv_x[];  // per vector two planes: elements 0-3 and 4-7 of every 8-element piece
  __shared__ float red[DGV_WARPS * NB];
  __shared__ float best_v[DGV_WARPS][NB];
  __shared__ int best_i[DGV_WARPS][NB];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int K = p.K, kc = pad8(K) >> 3, b0 = blockIdx.y * NB;
  pdl_launch_dependents();

  // ---- tasks: pairs of rows ----
  const int seg_fixed = p.ctas_per_seg ? (int)blockIdx.x / p.ctas_per_seg : -1;
  auto tasks_of = [&](int s) { return act_is_glu(p.seg[s].act) ? p.seg[s].rows : (p.seg[s].rows + 1) >> 1; };
  int ntasks = 0, task, stride;
  if (seg_fixed >= 0) {
    ntasks = tasks_of(seg_fixed);
    task = (blockIdx.x - seg_fixed * p.ctas_per_seg) * DGV_WARPS + warp;
    stride = p.ctas_per_seg * DGV_WARPS;
  } else {
    for (int s = 0; s < p.nseg; ++s) ntasks += tasks_of(s);
    task = blockIdx.x * DGV_WARPS + warp;
    stride = gridDim.x * DGV_WARPS;
  }
  int seg = 0, r0 = 0;  // of the current task
  bool has1 = false;    // the pair's second row exists
  const uint4 *w0 = nullptr, *w1 = nullptr;
  auto locate = [&](int t) {
    if (seg_fixed >= 0) seg = seg_fixed;
    else {
      seg = 0;
      while (seg + 1 < p.nseg && t >= tasks_of(seg)) { t -= tasks_of(seg); ++seg; }
    }
    const DgvSeg& sg = p.seg[seg];
    const bool glu = act_is_glu(sg.act);
    r0 = glu ? t : 2 * t;
    has1 = glu || r0 + 1 < sg.rows;
    const int64_t a = glu ? glu_row(r0, 0) : r0, b = glu ? glu_row(r0, 1) : (has1 ? r0 + 1 : r0);
    w0 = reinterpret_cast<const uint4*>(sg.w) + a * kc;
    w1 = reinterpret_cast<const uint4*>(sg.w) + b * kc;
  };
  uint4 wa[DGV_U], wb[DGV_U];
  auto load = [&](int it) {
#pragma unroll
    for (int u = 0; u < DGV_U; ++u) {
      const int c = (it * DGV_U + u) * 32 + lane;
      const bool ok = c < kc;
      wa[u] = ok ? ldg128(w0 + c) : make_uint4(0, 0, 0, 0);
      wb[u] = ok ? ldg128(w1 + c) : make_uint4(0, 0, 0, 0);
    }
  };
  if (task < ntasks) {
    locate(task);
    load(0);
  }
  pdl_wait();

  // ---- prologue ----
  const int n4 = 2 * kc;  // float4 pieces per vector
  auto slot_of = [&](int n) -> float4* { return reinterpret_cast<float4*>(dgv_x) + (size_t)n * n4; };
  auto place = [&](int j) { return (j & 1) * kc + (j >> 1); };  // float4 j of a vector -> its plane position
  float ss[NB];
  if (p.add && p.add_w) {
#pragma unroll
    for (int n = 0; n < NB; ++n) {
      ss[n] = 0.f;
      if (b0 + n < p.batch)
        for (int j = tid; j < n4; j += DGV_THREADS) {
          const float4 a = ld4_masked(p.add + (size_t)(b0 + n) * p.x_stride, 4 * j, K);
          ss[n] += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
        }
    }
    block_sums<NB, DGV_WARPS>(ss, red);
  }
  float sx[NB];
#pragma unroll
  for (int n = 0; n < NB; ++n) {
    sx[n] = 0.f;
    float4* dst = slot_of(n);
    if (b0 + n >= p.batch) {
      for (int j = tid; j < n4; j += DGV_THREADS) dst[place(j)] = make_float4(0.f, 0.f, 0.f, 0.f);
      continue;
    }
    const size_t row = (size_t)(b0 + n) * p.x_stride;
    const float f = p.add && p.add_w ? 1.0f / sqrtf(ss[n] / (float)K + p.eps) : 0.f;
    for (int j = tid; j < n4; j += DGV_THREADS) {
      float4 v = ld4_masked(p.x + row, 4 * j, K);
      if (p.add) {
        const float4 a = ld4_masked(p.add + row, 4 * j, K);
        if (p.add_w) {
          const float4 w = ld4_masked(p.add_w, 4 * j, K);
          v.x += a.x * f * w.x; v.y += a.y * f * w.y; v.z += a.z * f * w.z; v.w += a.w * f * w.w;
        } else {
          v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w;
        }
        if (p.add2) {
          const float4 e = ld4_masked(p.add2 + row, 4 * j, K);
          v.x += e.x; v.y += e.y; v.z += e.z; v.w += e.w;
        }
        if (blockIdx.x == 0) *reinterpret_cast<float4*>(p.x_out + row + 4 * j) = v;
      }
      dst[place(j)] = v;
      sx[n] += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  }
  if (p.norm_w) {
    block_sums<NB, DGV_WARPS>(sx, red);
    const float* mu = seg_fixed >= 0 ? p.seg[seg_fixed].mu : nullptr;
#pragma unroll
    for (int n = 0; n < NB; ++n) {
      if (b0 + n >= p.batch) continue;
      float4* dst = slot_of(n);
      const float f = 1.0f / sqrtf(sx[n] / (float)K + p.eps);
      const int pos = p.shift ? p.positions[b0 + n] : 0;
      float* hist = p.shift ? p.shift + (size_t)p.slots[b0 + n] * 2 * p.shift_stride : nullptr;
      for (int j = tid; j < n4; j += DGV_THREADS) {  // the same thread owns piece j in every pass
        float4 v = dst[place(j)];
        const float4 w = ld4_masked(p.norm_w, 4 * j, K);
        v.x *= f * w.x; v.y *= f * w.y; v.z *= f * w.z; v.w *= f * w.w;
        if (hist) {
          const float4 o = pos > 0 ? ld4_masked(hist + (size_t)(pos & 1) * p.shift_stride, 4 * j, K) : make_float4(0.f, 0.f, 0.f, 0.f);
          if (blockIdx.x == 0) *reinterpret_cast<float4*>(hist + (size_t)((pos + 1) & 1) * p.shift_stride + 4 * j) = v;
          const float4 m = ld4_masked(mu, 4 * j, K);
          v.x += (o.x - v.x) * m.x; v.y += (o.y - v.y) * m.y; v.z += (o.z - v.z) * m.z; v.w += (o.w - v.w) * m.w;
        }
        dst[place(j)] = v;
      }
    }
  }
  __syncthreads();

  // ---- rows ----
  const int my_row = lane & 1, my_col = lane >> 1;  // lanes 0 .. 2 NB - 1 finish one (row, vector) each
  float bv = -INFINITY;
  int bi = 0x7fffffff;
  const int iters = (kc + 32 * DGV_U - 1) / (32 * DGV_U);
  bool first = true;
  for (; task < ntasks; task += stride) {
    if (!first) locate(task);
    float acc[2][NB];
#pragma unroll
    for (int n = 0; n < NB; ++n) acc[0][n] = acc[1][n] = 0.f;
#pragma unroll 1
    for (int it = 0; it < iters; ++it) {
      if (!(first && it == 0)) load(it);
#pragma unroll
      for (int u = 0; u < DGV_U; ++u) {
        const int c = (it * DGV_U + u) * 32 + lane;
        if (c >= kc) continue;
        const uint4 a = wa[u], b = wb[u];
#pragma unroll
        for (int n = 0; n < NB; ++n) {
          const float4* xv = slot_of(n);
          const float4 lo = xv[c], hi = xv[kc + c];
          float s0 = acc[0][n], s1 = acc[1][n];
          s0 = fmaf(bf_lo(a.x), lo.x, s0); s1 = fmaf(bf_lo(b.x), lo.x, s1);
          s0 = fmaf(bf_hi(a.x), lo.y, s0); s1 = fmaf(bf_hi(b.x), lo.y, s1);
          s0 = fmaf(bf_lo(a.y), lo.z, s0); s1 = fmaf(bf_lo(b.y), lo.z, s1);
          s0 = fmaf(bf_hi(a.y), lo.w, s0); s1 = fmaf(bf_hi(b.y), lo.w, s1);
          s0 = fmaf(bf_lo(a.z), hi.x, s0); s1 = fmaf(bf_lo(b.z), hi.x, s1);
          s0 = fmaf(bf_hi(a.z), hi.y, s0); s1 = fmaf(bf_hi(b.z), hi.y, s1);
          s0 = fmaf(bf_lo(a.w), hi.z, s0); s1 = fmaf(bf_lo(b.w), hi.z, s1);
          s0 = fmaf(bf_hi(a.w), hi.w, s0); s1 = fmaf(bf_hi(b.w), hi.w, s1);
          acc[0][n] = s0; acc[1][n] = s1;
        }
      }
    }
    first = false;
    float mine = 0.f, pair = 0.f;  // this lane's (row, vector) sum, and the pair's second row
#pragma unroll
    for (int n = 0; n < NB; ++n) {
      const float t0 = warp_sum(acc[0][n]), t1 = warp_sum(acc[1][n]);
      if (my_col == n) { mine = my_row ? t1 : t0; pair = t1; }
    }
    const int b = b0 + my_col;
    if (my_col < NB && b < p.batch) {
      const DgvSeg& sg = p.seg[seg];
      if (act_is_glu(sg.act)) {
        if (my_row == 0) sg.y[(size_t)b * sg.y_stride + r0] = glu_act(sg.act, mine, pair);
      } else if (my_row == 0 || has1) {
        const int row = r0 + my_row;
        float v = dense_act(sg.act, sg.bias ? mine + sg.bias[row] : mine, sg.arg);
        if (p.pen_counts) {
          const int times = p.pen_counts[(size_t)b * p.pen_stride + row];
          const float pen = *p.pen_value;
          for (int i = 0; i < times; ++i) v = v > 0.f ? v / pen : v * pen;
        }
        sg.y[(size_t)b * sg.y_stride + row] = v;
        if (v > bv) { bv = v; bi = row; }
      }
    }
  }
  if (p.amax_val) {
    const float ov = __shfl_xor_sync(0xffffffffu, bv, 1);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, 1);
    if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
    if (my_row == 0 && my_col < NB) { best_v[warp][my_col] = bv; best_i[warp][my_col] = bi; }
    __syncthreads();
    if (tid < NB && b0 + tid < p.batch) {
      float v = best_v[0][tid];
      int i = best_i[0][tid];
      for (int w = 1; w < DGV_WARPS; ++w)
        if (best_v[w][tid] > v || (best_v[w][tid] == v && best_i[w][tid] < i)) { v = best_v[w][tid]; i = best_i[w][tid]; }
      p.amax_val[(size_t)(b0 + tid) * gridDim.x + blockIdx.x] = v;
      p.amax_idx[(size_t)(b0 + tid) * gridDim.x + blockIdx.x] = i;
    }
  }
}

}  // namespace b200
