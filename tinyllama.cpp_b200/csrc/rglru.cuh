// RG-LRU mixer: a gated linear recurrence per channel behind a short causal convolution. With x and y the two projections of
// the layer's input (y through its activation already):
//   u_t = sum_k conv[k] x_(t - taps + 1 + k) + conv_b                   (zeros before the start)
//   r_t = sigmoid(R u_t + r_b), i_t = sigmoid(I u_t + i_b)              (R, I block-diagonal)
//   a_t = exp(-8 r_t softplus(lam)),  S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t,  output S_t * y_t
// Everything here is FP32; the gate products of prompts run on the tensor cores with u as the sum of two bfloat16 numbers
// (value and remainder) against the bfloat16 weights, or, in a 32-bit engine, as plain FP32 arithmetic.
//
//   rglru_step_kernel   one token of several sequences (decode): convolution, gates, recurrence and the product with y
//   rglru_gates_kernel  prompts: 64 tokens x 64 channels per block; convolution and gates, then the recurrence inside the
//                       tile as pairs (P, Q) with S_t = P_t S_(tile start) + Q_t
//   rglru_apply_kernel  prompts: the state at every tile's start from the tiles before it, then S_t * y_t; stores the state
//
// State of a slot: S [width], and the convolution's last inputs as a ring [taps][width] (position p in row p % taps). A
// token at position 0 starts from zeros whatever the slot held before.
#pragma once
#include "attn_tiles.cuh"

namespace b200 {

struct RgLruParams {
  const float* x;          // [T][stride] the branch that goes through the convolution
  const float* y;          // [T][stride] the other one, activated
  int stride;
  const float* conv;       // [taps][wp]: row k multiplies the input taps - 1 - k tokens back
  const float* conv_b;     // [width]
  int taps;
  const __nv_bfloat16 *ra, *ri;  // [width][pad8(bs)]: row c of block c / bs
  const float *ra_b, *ri_b;
  const float* decay;      // [width]: 8 softplus(lam)
  float* state;            // [slot][wp]
  float* ring;             // [slot][taps][wp]
  int width, wp, blocks, bs;  // bs = width / blocks
  // decode
  const int* positions;
  const int* slots;
  int batch;
  // prompts
  const RunDesc* runs;
  float *P, *Q;            // [T][pq_stride]
  int pq_stride;
  void* out;               // [T][out_stride]
  int out_stride;
};

__device__ __forceinline__ float gate_sigmoid(float z) { return rcp_fast(1.0f + ex2_fast(-1.4426950408889634f * z)); }
// a and sqrt(1 - a^2) from the gate's product r (before the sigmoid). 1 - a^2 = 1 - e^x with x = 2 log a loses digits for
// small x: there it is -x times the series of (e^x - 1) / x.
__device__ __forceinline__ void rglru_decay(float r, float decay, float& a, float& norm) {
  const float log_a = -decay * gate_sigmoid(r), x = 2.0f * log_a;
  a = ex2_fast(1.4426950408889634f * log_a);
  float series = fmaf(x, 1.f / 5040.f, 1.f / 720.f);
  series = fmaf(x, series, 1.f / 120.f);
  series = fmaf(x, series, 1.f / 24.f);
  series = fmaf(x, series, 1.f / 6.f);
  series = fmaf(x, series, 0.5f);
  series = fmaf(x, series, 1.f);
  const float left = x > -0.5f ? -x * series : fmaf(-a, a, 1.f);
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(norm) : "f"(left));
}

// Sums N values over the warp (N a power of two up to 32): every lane gets the total of value lane % N.
template <int N>
__device__ __forceinline__ float lane_sums(float (&v)[N]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int s = N / 2; s > 0; s >>= 1)
#pragma unroll
    for (int j = 0; j < s; ++j) {
      const bool up = lane & s;
      const float send = up ? v[j] : v[j + s], keep = up ? v[j + s] : v[j];
      v[j] = keep + __shfl_xor_sync(0xffffffffu, send, s);
    }
#pragma unroll
  for (int s = N; s < 32; s <<= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], s);
  return v[0];
}

constexpr int RGS_THREADS = 256, RGS_WARPS = 8;
constexpr int RGS_ROWS = 4;                        // channels per warp
constexpr int RGS_CH = RGS_WARPS * RGS_ROWS;       // channels per block
constexpr size_t RGS_SMEM_MAX = 96 * 1024;

__host__ __device__ __forceinline__ size_t rgs_smem_bytes(int bs, int nb) { return (size_t)nb * pad8(bs) * 4; }

// grid = (blocks * pieces of 32 channels, batch / NB rounded up). Every block forms u of its whole gate block.
template <int NB, typename O>
__global__ void __launch_bounds__(RGS_THREADS) rglru_step_kernel(const RgLruParams p) {
  extern __shared__ __align__(16) float rgs_u[];  // [NB][pad8(bs)]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, kc = pad8(p.bs) >> 3, up = 8 * kc;
  const int pieces = (p.bs + RGS_CH - 1) / RGS_CH, blk = blockIdx.x / pieces, piece = blockIdx.x - blk * pieces;
  const int b0 = blockIdx.y * NB, nb = min(NB, p.batch - b0), base = blk * p.bs, c0 = piece * RGS_CH + warp * RGS_ROWS;
  pdl_launch_dependents();
  // this warp's rows of both gate matrices: 16-byte pieces, requested before anything else
  uint4 w[2][RGS_ROWS];
  auto load = [&](int it) {
    const int c = it * 32 + lane;
#pragma unroll
    for (int i = 0; i < RGS_ROWS; ++i) {
      const bool ok = c < kc && c0 + i < p.bs;
      const size_t at = (size_t)(base + c0 + i) * kc + c;
      w[0][i] = ok ? ldg128(reinterpret_cast<const uint4*>(p.ra) + at) : make_uint4(0, 0, 0, 0);
      w[1][i] = ok ? ldg128(reinterpret_cast<const uint4*>(p.ri) + at) : make_uint4(0, 0, 0, 0);
    }
  };
  load(0);
  pdl_wait();
  // what this lane finishes: channel (lane % 4) of sequence lane / 4
  const int fn = lane / RGS_ROWS, fc = c0 + lane % RGS_ROWS, fch = base + fc;
  const bool mine = fn < nb && fc < p.bs;
  float old = 0.f, yv = 0.f, rb = 0.f, ib = 0.f, dec = 0.f;
  float* S = nullptr;
  if (mine) {
    S = p.state + (size_t)p.slots[b0 + fn] * p.wp + fch;
    if (p.positions[b0 + fn] > 0) old = *S;
    yv = p.y[(size_t)(b0 + fn) * p.stride + fch];
    rb = p.ra_b[fch]; ib = p.ri_b[fch]; dec = p.decay[fch];
  }
  int pos[NB];
  float* ring[NB];
#pragma unroll
  for (int n = 0; n < NB; ++n) {
    pos[n] = n < nb ? p.positions[b0 + n] : 0;
    ring[n] = p.ring + (n < nb ? (size_t)p.slots[b0 + n] * p.taps * p.wp : 0) + base;
  }
  for (int c = tid; c < up; c += RGS_THREADS) {
    const bool ok = c < p.bs;
    const int ch = base + (ok ? c : 0);
    const float w = p.conv[(size_t)(p.taps - 1) * p.wp + ch], bias = p.conv_b[ch];
    float u[NB];
#pragma unroll
    for (int n = 0; n < NB; ++n) {
      const float x = ok && n < nb ? p.x[(size_t)(b0 + n) * p.stride + ch] : 0.f;
      u[n] = fmaf(w, x, bias);
      if (piece == 0 && ok && n < nb) ring[n][(size_t)(pos[n] % p.taps) * p.wp + c] = x;  // a row nobody reads in this launch
    }
    for (int k = 1; k < p.taps; ++k) {
      const float wk = p.conv[(size_t)(p.taps - 1 - k) * p.wp + ch];
#pragma unroll
      for (int n = 0; n < NB; ++n)
        if (ok && k <= pos[n]) u[n] = fmaf(wk, ring[n][(size_t)((pos[n] - k) % p.taps) * p.wp + c], u[n]);
    }
#pragma unroll
    for (int n = 0; n < NB; ++n) rgs_u[n * up + c] = ok && n < nb ? u[n] : 0.f;
  }
  __syncthreads();
  float acc[2][RGS_ROWS * NB];  // [matrix][sequence * 4 + channel]
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int i = 0; i < RGS_ROWS * NB; ++i) acc[m][i] = 0.f;
  for (int it = 0; it * 32 < kc; ++it) {
    if (it) load(it);
    const int c = it * 32 + lane;
    if (c >= kc) continue;
#pragma unroll
    for (int n = 0; n < NB; ++n) {
      float u[8];
      load8(rgs_u + n * up + 8 * c, u);
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int i = 0; i < RGS_ROWS; ++i) {
          const uint4 v = w[m][i];
          float s = acc[m][n * RGS_ROWS + i];
          s = fmaf(bf_lo(v.x), u[0], s); s = fmaf(bf_hi(v.x), u[1], s); s = fmaf(bf_lo(v.y), u[2], s); s = fmaf(bf_hi(v.y), u[3], s);
          s = fmaf(bf_lo(v.z), u[4], s); s = fmaf(bf_hi(v.z), u[5], s); s = fmaf(bf_lo(v.w), u[6], s); s = fmaf(bf_hi(v.w), u[7], s);
          acc[m][n * RGS_ROWS + i] = s;
        }
    }
  }
  const float r = lane_sums(acc[0]), g = lane_sums(acc[1]);
  if (!mine) return;
  float a, norm;
  rglru_decay(r + rb, dec, a, norm);
  const float s = fmaf(a, old, norm * gate_sigmoid(g + ib) * rgs_u[fn * up + fc]);
  *S = s;
  static_cast<O*>(p.out)[(size_t)(b0 + fn) * p.out_stride + fch] = to_operand<O>(s * yv);
}

// ---- prompts -----------------------------------------------------------------------------------------------------
constexpr int RGP_TILE = 64;                     // tokens and channels of a block, columns of a K step
constexpr int RGP_THREADS = 256;
constexpr int RGP_LD = RGP_TILE + 8;             // row stride of the operand tiles (bfloat16)
constexpr int RGP_STAGE = 4 * RGP_TILE * RGP_LD * 2;  // R | I | u (value, remainder; or FP32)
constexpr int RGP_FLD = RGP_TILE + 1;            // row stride of the FP32 tiles [token][channel]
constexpr size_t RGP_SMEM = 2 * RGP_STAGE + (size_t)RGP_TILE * RGP_FLD * 4;
constexpr int RGP_SEG = RGP_TILE / (RGP_THREADS / RGP_TILE);  // tokens per thread of the scan and of the convolution
constexpr int RGP_TAPS = 4;                      // taps the register window of the convolution covers

// grid = (64-token tiles of the longest run, blocks * pieces of 64 channels, runs). F32: FP32 products.
template <bool F32>
__global__ void __launch_bounds__(RGP_THREADS) rglru_gates_kernel(const RgLruParams p) {
  extern __shared__ __align__(16) unsigned char rgp_smem[];
  __shared__ float seg_p[RGP_THREADS], seg_q[RGP_THREADS];
  const RunDesc run = p.runs[blockIdx.z];
  const int t0 = blockIdx.x * RGP_TILE;
  if (t0 >= run.len) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nt = min(RGP_TILE, run.len - t0);
  const int pieces = (p.bs + RGP_TILE - 1) / RGP_TILE, blk = blockIdx.y / pieces, piece = blockIdx.y - blk * pieces;
  const int base = blk * p.bs, c0 = piece * RGP_TILE, ld = pad8(p.bs), steps = pieces;
  float* Us = reinterpret_cast<float*>(rgp_smem + 2 * RGP_STAGE);  // u of this block's channels, [token][channel]
  const float* ring = p.ring + (size_t)run.slot * p.taps * p.wp;

  // ---- operand tiles ----
  auto fetch_w = [&](int step) {
    __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(rgp_smem + (step & 1) * RGP_STAGE);
    for (int i = tid; i < 2 * RGP_TILE * (RGP_TILE / 8); i += RGP_THREADS) {
      const int m = i / (RGP_TILE * (RGP_TILE / 8)), r = i / (RGP_TILE / 8) % RGP_TILE, c = i % (RGP_TILE / 8) * 8, k = step * RGP_TILE + c;
      __nv_bfloat16* d = dst + (m * RGP_TILE + r) * RGP_LD + c;
      if (c0 + r < p.bs && k < ld) pfa_cp16(d, (m ? p.ri : p.ra) + (size_t)(base + c0 + r) * ld + k);
      else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // this thread's share of the convolution: one channel, RGP_SEG consecutive tokens
  const int cc = tid % RGP_TILE, ct = tid / RGP_TILE * RGP_SEG;
  auto before = [&](int ch, int t) {  // x of token t < 0 of the run
    const int pos = run.start + t;
    return pos >= 0 ? ring[(size_t)(pos % p.taps) * p.wp + ch] : 0.f;
  };
  const float* xs = p.x + (size_t)(run.row0 + t0 + ct) * p.stride;
  const int left = run.len - t0 - ct;  // tokens of the run from this thread's first one on
  float win[RGP_SEG + RGP_TAPS - 1];   // win[j]: token j - (RGP_TAPS - 1) from there
  auto fetch_x = [&](int step) {
    const int c = step * RGP_TILE + cc, ch = base + c;
    const bool ok = c < p.bs;
#pragma unroll
    for (int j = 0; j < RGP_SEG; ++j) win[RGP_TAPS - 1 + j] = ok && j < left ? xs[(size_t)j * p.stride + ch] : 0.f;
#pragma unroll
    for (int back = 1; back < RGP_TAPS; ++back) {  // tokens further back than the taps reach are not kept
      float v = 0.f;
      if (ok && left > 0 && back < p.taps) v = t0 + ct >= back ? xs[ch - (ptrdiff_t)back * p.stride] : before(ch, t0 + ct - back);
      win[RGP_TAPS - 1 - back] = v;
    }
  };
  auto store_u = [&](int step) {
    const int c = step * RGP_TILE + cc, ch = base + c;
    unsigned char* stage = rgp_smem + (step & 1) * RGP_STAGE + 2 * RGP_TILE * RGP_LD * 2;
    __nv_bfloat16 *hi = reinterpret_cast<__nv_bfloat16*>(stage), *lo = hi + RGP_TILE * RGP_LD;
    float* f = reinterpret_cast<float*>(stage);
    const bool ok = c < p.bs;
    const float bias = ok ? p.conv_b[ch] : 0.f;
    auto put = [&](int j, float u) {
      if (F32) f[(ct + j) * RGP_LD + cc] = u;
      else split_bf16(u, hi[(ct + j) * RGP_LD + cc], lo[(ct + j) * RGP_LD + cc]);
      if (step == piece) Us[(ct + j) * RGP_FLD + cc] = u;
    };
    if (p.taps > RGP_TAPS) {  // any number of taps, straight from memory
#pragma unroll 1
      for (int j = 0; j < RGP_SEG; ++j) {
        float u = bias;
        if (ok && j < left)
          for (int k = 0; k < p.taps; ++k) {
            const float x = t0 + ct + j >= k ? xs[ch + (ptrdiff_t)(j - k) * p.stride] : before(ch, t0 + ct + j - k);
            u = fmaf(p.conv[(size_t)(p.taps - 1 - k) * p.wp + ch], x, u);
          }
        put(j, u);
      }
      return;
    }
    float w[RGP_TAPS];
#pragma unroll
    for (int k = 0; k < RGP_TAPS; ++k) w[k] = ok && k < p.taps ? p.conv[(size_t)(p.taps - 1 - k) * p.wp + ch] : 0.f;  // k tokens back
#pragma unroll
    for (int j = 0; j < RGP_SEG; ++j) {  // values of tokens beyond the run stay unused
      float u = bias;
#pragma unroll
      for (int k = 0; k < RGP_TAPS; ++k) u = fmaf(w[k], win[j + RGP_TAPS - 1 - k], u);
      put(j, u);
    }
  };

  // ---- gate products: 16 channels x 32 tokens of both matrices per warp ----
  const int r0 = 16 * (warp & 3), n0 = 32 * (warp >> 2), g = lane >> 2, t = lane & 3;
  float acc[2][4][4];
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[m][i][0] = acc[m][i][1] = acc[m][i][2] = acc[m][i][3] = 0.f;
  fetch_w(0);
  fetch_x(0);
  store_u(0);
  for (int step = 0; step < steps; ++step) {
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();  // the stage is complete, and everyone has left the other one
    if (step + 1 < steps) {
      fetch_w(step + 1);
      fetch_x(step + 1);
    }
    const __nv_bfloat16* ws = reinterpret_cast<const __nv_bfloat16*>(rgp_smem + (step & 1) * RGP_STAGE);
    if (F32) {
      const float* us = reinterpret_cast<const float*>(ws + 2 * RGP_TILE * RGP_LD);
      for (int k = 0; k < RGP_TILE; ++k) {
        float w[2][2];
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int e = 0; e < 2; ++e) w[m][e] = __bfloat162float(ws[(m * RGP_TILE + r0 + g + 8 * e) * RGP_LD + k]);
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float u = us[(n0 + 8 * i + 2 * t + e) * RGP_LD + k];
#pragma unroll
            for (int m = 0; m < 2; ++m) {
              acc[m][i][e] = fmaf(w[m][0], u, acc[m][i][e]);
              acc[m][i][2 + e] = fmaf(w[m][1], u, acc[m][i][2 + e]);
            }
          }
      }
    } else {
      const __nv_bfloat16* us = ws + 2 * RGP_TILE * RGP_LD;
#pragma unroll
      for (int ks = 0; ks < RGP_TILE; ks += 16) {
        uint32_t a[2][4];
#pragma unroll
        for (int m = 0; m < 2; ++m) pfa_ldm4(a[m], ws + (m * RGP_TILE + r0 + (lane & 15)) * RGP_LD + ks + (lane >> 4) * 8);
#pragma unroll
        for (int half = 0; half < 2; ++half)  // values, then remainders
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            uint32_t b[4];
            pfa_ldm4(b, us + (half * RGP_TILE + n0 + i * 16 + (lane & 7) + (lane >> 4) * 8) * RGP_LD + ks + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int m = 0; m < 2; ++m) {
              lap_mma(acc[m][2 * i], a[m], b[0], b[1]);
              lap_mma(acc[m][2 * i + 1], a[m], b[2], b[3]);
            }
          }
      }
    }
    if (step + 1 < steps) store_u(step + 1);
  }
  __syncthreads();  // the operand tiles are free, u is complete

  // ---- recurrence inside the tile: 16 tokens of a channel per thread, then the segments before this one ----
  float *Rs = reinterpret_cast<float*>(rgp_smem), *Is = Rs + RGP_TILE * RGP_FLD;  // gate products [token][channel]
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int at = (n0 + 8 * i + 2 * t + (e & 1)) * RGP_FLD + r0 + g + 8 * (e >> 1);
      Rs[at] = acc[0][i][e];
      Is[at] = acc[1][i][e];
    }
  __syncthreads();
  const int last = min(ct + RGP_SEG, nt);
  const bool mine = c0 + cc < p.bs;
  const int ch = base + c0 + (mine ? cc : 0);
  const float rb = p.ra_b[ch], ib = p.ri_b[ch], dec = p.decay[ch];
  float P = 1.f, Q = 0.f;
#pragma unroll 2
  for (int j = ct; j < last; ++j) {  // the pair of every token, in place of its gate product and u
    const int at = j * RGP_FLD + cc;
    float a, norm;
    rglru_decay(Rs[at] + rb, dec, a, norm);
    P *= a;
    Q = fmaf(a, Q, norm * gate_sigmoid(Is[at] + ib) * Us[at]);
    Rs[at] = P;
    Us[at] = Q;
  }
  seg_p[tid] = P;
  seg_q[tid] = Q;
  __syncthreads();
  if (!mine) return;
  P = 1.f;
  Q = t0 == 0 && run.start > 0 ? p.state[(size_t)run.slot * p.wp + ch] : 0.f;  // the run's first tile starts from the slot's state
  for (int s = cc; s < tid; s += RGP_TILE) {
    Q = fmaf(seg_p[s], Q, seg_q[s]);
    P *= seg_p[s];
  }
#pragma unroll 4
  for (int j = ct; j < last; ++j) {
    const size_t row = (size_t)(run.row0 + t0 + j) * p.pq_stride + ch;
    const float pj = Rs[j * RGP_FLD + cc];
    p.P[row] = P * pj;
    p.Q[row] = fmaf(pj, Q, Us[j * RGP_FLD + cc]);
  }
}

constexpr int RGA_THREADS = 128, RGA_TOKENS = 16;  // channels and tokens of a block

// grid = (16-token pieces of the longest run, 128-channel pieces, runs). The last row of a tile holds the pair of the whole
// tile; the first tile's rows are the states themselves.
template <typename O>
__global__ void __launch_bounds__(RGA_THREADS) rglru_apply_kernel(const RgLruParams p) {
  const RunDesc run = p.runs[blockIdx.z];
  const int t0 = blockIdx.x * RGA_TOKENS, ch = blockIdx.y * RGA_THREADS + threadIdx.x;
  if (t0 >= run.len || ch >= p.width) return;
  const float *P = p.P + (size_t)run.row0 * p.pq_stride + ch, *Q = p.Q + (size_t)run.row0 * p.pq_stride + ch;
  float S = 0.f;
  const int tiles = t0 / RGP_TILE;
#pragma unroll 8
  for (int i = 0; i < tiles; ++i) {
    const size_t last = (size_t)(i * RGP_TILE + RGP_TILE - 1) * p.pq_stride;
    S = i ? fmaf(P[last], S, Q[last]) : Q[last];
  }
  const int n = min(RGA_TOKENS, run.len - t0);
  const float* y = p.y + (size_t)(run.row0 + t0) * p.stride + ch;
  O* out = static_cast<O*>(p.out) + (size_t)(run.row0 + t0) * p.out_stride + ch;
  P += (size_t)t0 * p.pq_stride;
  Q += (size_t)t0 * p.pq_stride;
  float s = 0.f;
#pragma unroll 8
  for (int j = 0; j < n; ++j) {
    s = tiles ? fmaf(P[(size_t)j * p.pq_stride], S, Q[(size_t)j * p.pq_stride]) : Q[(size_t)j * p.pq_stride];
    out[(size_t)j * p.out_stride] = to_operand<O>(s * y[(size_t)j * p.stride]);
  }
  if (t0 + n == run.len) p.state[(size_t)run.slot * p.wp + ch] = s;
  for (int j = max(0, run.len - p.taps - t0); j < n; ++j)  // the inputs the next convolution looks back at
    p.ring[((size_t)run.slot * p.taps + (run.start + t0 + j) % p.taps) * p.wp + ch] = p.x[(size_t)(run.row0 + t0 + j) * p.stride + ch];
}

}  // namespace b200
