// Row kernels of the block models' prompt path (many tokens per launch): embedding, the norms between sublayers, the
// token-shift mixes, the head norm of the WKV mixer. Each writes the operand type of the next matmul: A = __nv_bfloat16
// or, in a 32-bit engine, float. Norms and the residual stream are FP32 throughout.
#pragma once
#include "dense_gemv.cuh"

namespace b200 {

// A run of consecutive tokens of one sequence inside a chunk, as the kernels see it.
struct RunDesc {
  int row0, len, slot, start;  // rows of the chunk, KV slot, position of the first token
  int ctx0, hist;              // latent attention: first row of the run in the expanded context, cached rows before the run
};

template <typename A>
__device__ __forceinline__ A to_operand(float v);
template <>
__device__ __forceinline__ float to_operand<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 to_operand<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// x[b][:] = table[tokens[b]][:] * scale, and the same into `again` if given. grid.x = tokens.
__global__ void embed_bf16_kernel(const int* __restrict__ tokens, const __nv_bfloat16* __restrict__ table, int ld, float scale, float* __restrict__ x,
                                  float* __restrict__ again, int x_stride, int W, int vocab) {
  const int b = blockIdx.x;
  const int tok = min(max(tokens[b], 0), vocab - 1);
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    const float v = __bfloat162float(table[(size_t)tok * ld + i]) * scale;
    x[(size_t)b * x_stride + i] = v;
    if (again) again[(size_t)b * x_stride + i] = v;
  }
}

constexpr int ROW_THREADS = 256;

struct NormRowsParams {
  float* x;            // [T][x_stride] residual stream, updated in place when `add` is given
  int x_stride, W;
  const float* add;    // pending sublayer output [T][x_stride]
  const float* add_w;  // its norm, or nullptr: added as it is
  const float* add2;   // further rows added to the stream [T][x_stride] (only with add), or nullptr
  const float* norm_w; // nullptr: only the residual update
  float eps;
  const int* gather;   // row i of the output comes from row gather[i] of x (x itself is left as it is then)
  float* h32;          // optional FP32 copy of the normalised rows [T][x_stride]
  void* out;           // [T][out_stride] operand rows, optional
  int out_stride;
};

// One block per row: x += rms(add) * add_w (or add), x += add2; out = rms(x) * norm_w.
template <typename A>
__global__ void __launch_bounds__(ROW_THREADS) norm_rows_kernel(const NormRowsParams p) {
  extern __shared__ __align__(16) float row_s[];
  __shared__ float red[ROW_THREADS / 32];
  const int tid = threadIdx.x, n4 = pad8(p.W) >> 2;
  const size_t src = p.gather ? (size_t)p.gather[blockIdx.x] : blockIdx.x;
  float* xr = p.x + src * p.x_stride;
  float4* s4 = reinterpret_cast<float4*>(row_s);
  float f = 0.f, ss[1];
  const float* ar = p.add ? p.add + src * p.x_stride : nullptr;
  if (ar && p.add_w) {
    ss[0] = 0.f;
    for (int j = tid; j < n4; j += ROW_THREADS) {
      const float4 a = ld4_masked(ar, 4 * j, p.W);
      s4[j] = a;
      ss[0] += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
    }
    block_sums<1, ROW_THREADS / 32>(ss, red);
    f = 1.0f / sqrtf(ss[0] / (float)p.W + p.eps);
  }
  ss[0] = 0.f;
  for (int j = tid; j < n4; j += ROW_THREADS) {
    float4 v = ld4_masked(xr, 4 * j, p.W);
    if (ar) {
      if (p.add_w) {
        const float4 a = s4[j], w = ld4_masked(p.add_w, 4 * j, p.W);
        v.x += a.x * f * w.x; v.y += a.y * f * w.y; v.z += a.z * f * w.z; v.w += a.w * f * w.w;
      } else {
        const float4 a = ld4_masked(ar, 4 * j, p.W);
        v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w;
      }
      if (p.add2) {
        const float4 e = ld4_masked(p.add2 + src * p.x_stride, 4 * j, p.W);
        v.x += e.x; v.y += e.y; v.z += e.z; v.w += e.w;
      }
      if (!p.gather) *reinterpret_cast<float4*>(xr + 4 * j) = v;
    }
    s4[j] = v;
    ss[0] += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  if (!p.norm_w) return;
  block_sums<1, ROW_THREADS / 32>(ss, red);
  f = 1.0f / sqrtf(ss[0] / (float)p.W + p.eps);
  for (int j = tid; j < n4; j += ROW_THREADS) {
    float4 v = s4[j];
    const float4 w = ld4_masked(p.norm_w, 4 * j, p.W);
    v.x *= f * w.x; v.y *= f * w.y; v.z *= f * w.z; v.w *= f * w.w;
    if (p.h32) *reinterpret_cast<float4*>(p.h32 + (size_t)blockIdx.x * p.x_stride + 4 * j) = v;
    if (p.out) {
      A* o = static_cast<A*>(p.out) + (size_t)blockIdx.x * p.out_stride + 4 * j;
      o[0] = to_operand<A>(v.x); o[1] = to_operand<A>(v.y); o[2] = to_operand<A>(v.z); o[3] = to_operand<A>(v.w);
    }
  }
}

// RMS norm of the first n elements of each row into an operand row (the query latent). grid.x = rows.
template <typename A>
__global__ void __launch_bounds__(ROW_THREADS) norm_head_rows_kernel(const float* __restrict__ x, int x_stride, int n, const float* __restrict__ w, float eps,
                                                                     A* __restrict__ out, int out_stride) {
  __shared__ float red[ROW_THREADS / 32];
  const float* xr = x + (size_t)blockIdx.x * x_stride;
  float ss[1] = {0.f};
  for (int i = threadIdx.x; i < n; i += ROW_THREADS) ss[0] += xr[i] * xr[i];
  block_sums<1, ROW_THREADS / 32>(ss, red);
  const float f = 1.0f / sqrtf(ss[0] / (float)n + eps);
  for (int i = threadIdx.x; i < n; i += ROW_THREADS) out[(size_t)blockIdx.x * out_stride + i] = to_operand<A>(xr[i] * f * w[i]);
}

struct MixRowsParams {
  const float* h;        // [T][h_stride] normalised rows
  int h_stride, W, nruns;
  const RunDesc* runs;   // runs of the chunk in row order; nullptr: every row is a token of its own (slots, positions)
  const int* slots;
  const int* positions;
  const float* shift;    // [slot][2][shift_stride]
  int shift_stride;
  const float* mu[5];
  void* out[5];          // operand rows [T][out_stride]
  int out_stride;
};

// The run that holds row t.
__device__ __forceinline__ int run_of_row(const RunDesc* runs, int nruns, int t) {
  int lo = 0, hi = nruns - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (runs[mid].row0 <= t) lo = mid;
    else hi = mid - 1;
  }
  return lo;
}

// Token shift: five mixes of every row with the row of the previous token (the slot's saved row at the start of a run,
// zeros at position 0). With runs == nullptr the row itself is saved as the next step's previous row.
template <typename A>
__global__ void __launch_bounds__(ROW_THREADS) mix_rows_kernel(const MixRowsParams p, float* shift_out) {
  const int t = blockIdx.x;
  const float* hr = p.h + (size_t)t * p.h_stride;
  const float* prev = nullptr;
  float* save = nullptr;
  if (p.runs) {
    const RunDesc r = p.runs[run_of_row(p.runs, p.nruns, t)];
    if (t > r.row0) prev = hr - p.h_stride;
    else if (r.start > 0) prev = p.shift + ((size_t)r.slot * 2 + (r.start & 1)) * p.shift_stride;
  } else {
    const int pos = p.positions[t], slot = p.slots[t];
    if (pos > 0) prev = p.shift + ((size_t)slot * 2 + (pos & 1)) * p.shift_stride;
    save = shift_out + ((size_t)slot * 2 + ((pos + 1) & 1)) * p.shift_stride;
  }
  for (int i = threadIdx.x; i < p.W; i += ROW_THREADS) {
    const float h = hr[i], d = (prev ? prev[i] : 0.f) - h;
#pragma unroll
    for (int s = 0; s < 5; ++s) static_cast<A*>(p.out[s])[(size_t)t * p.out_stride + i] = to_operand<A>(h + d * p.mu[s][i]);
    if (save) save[i] = h;
  }
}

// Per head: o / rms(o), times the norm weight and the gate. One warp per (row, head).
template <typename A>
__global__ void __launch_bounds__(ROW_THREADS) head_norm_gate_kernel(const float* __restrict__ o, int o_stride, const float* __restrict__ gate, int gate_stride,
                                                                     const float* __restrict__ w, int heads, int dim, float eps, int T, A* __restrict__ out,
                                                                     int out_stride) {
  const int item = blockIdx.x * (ROW_THREADS / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= T * heads) return;
  const int t = item / heads, h = item - t * heads;
  const float* r = o + (size_t)t * o_stride + h * dim;
  float ss = 0.f;
  for (int i = lane; i < dim; i += 32) ss += r[i] * r[i];
  const float f = 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps);
  for (int i = lane; i < dim; i += 32)
    out[(size_t)t * out_stride + h * dim + i] = to_operand<A>(r[i] * f * w[h * dim + i] * gate[(size_t)t * gate_stride + h * dim + i]);
}

}  // namespace b200
