// WKV mixer: the recurrence S <- diag(w_t) S + k_t v_t^T per head (S is key x value, FP32), read out before the update
// with a bonus for the current token: o_t = (S + diag(u) k_t v_t^T)^T r_t. Everything here is FP32.
//
//   wkv_step_kernel  one token of several sequences (decode): one block per (head, sequence); the decay's second matrix
//                    product, the recurrence, the head norm and the gate in one launch
//   wkv_scan_kernel  runs of tokens (prompts): the value columns of a head are independent of one another, so a block
//                    takes a few columns of one head, keeps their state in registers (four or eight keys of two columns per thread) and walks
//                    the run's tokens, whose r, k, w, v pieces arrive in shared memory a tile ahead (cp.async)
//
// State of a slot: [head][key][value]. A token at position 0 starts from zeros whatever the slot held before.
#pragma once
#include <type_traits>

#include "block_rows.cuh"

namespace b200 {

constexpr int WKV_STEP_THREADS = 256;
constexpr int WKV_MAX_DIM = 256;

struct WkvStepParams {
  const float* rkvg;      // [batch][stride]: r, k, v, gate at offsets 0, hd, 2 hd, 3 hd (hd = padded heads * dim)
  int stride, off;        // off = hd
  const float* low;       // [batch][low_stride] inner vector of the decay product
  int low_stride, rank;
  const __nv_bfloat16* w2;  // [heads * dim][pad8(rank)]
  const float* w0;
  const float* u;
  const float* norm;
  float eps;
  float* state;           // [slot][heads][dim][dim]
  const int* slots;
  const int* positions;
  int heads, dim;
  void* out;              // [batch][out_stride]
  int out_stride;
};

template <typename A>
__global__ void __launch_bounds__(WKV_STEP_THREADS) wkv_step_kernel(const WkvStepParams p) {
  __shared__ float r_s[WKV_MAX_DIM], k_s[WKV_MAX_DIM], w_s[WKV_MAX_DIM], part[WKV_STEP_THREADS], red[WKV_STEP_THREADS / 32];
  const int tid = threadIdx.x, h = blockIdx.x, b = blockIdx.y, D = p.dim, hc = h * D;
  pdl_launch_dependents();
  constexpr int W2_KEEP = 8;  // pieces of the decay row requested ahead (rank up to 64)
  const int rp = pad8(p.rank) >> 3;
  const uint4* w2 = reinterpret_cast<const uint4*>(p.w2) + (size_t)(hc + min(tid, D - 1)) * rp;
  uint4 wk[W2_KEEP];
#pragma unroll
  for (int i = 0; i < W2_KEEP; ++i) wk[i] = tid < D && i < rp ? ldg128(w2 + i) : make_uint4(0, 0, 0, 0);
  pdl_wait();
  const float* in = p.rkvg + (size_t)b * p.stride + hc;
  const int pos = p.positions[b];
  float* S = p.state + ((size_t)p.slots[b] * p.heads + h) * D * D;
  const int groups = WKV_STEP_THREADS / D;  // key groups working side by side on every value column
  const int col = tid % D, grp = tid / D;
  const bool active = grp < groups;
  constexpr int KEEP = 16;  // state elements per thread held in registers (all of them up to dim 64)
  float st[KEEP];
  if (active && pos > 0) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int k = grp + i * groups;
      st[i] = k < D ? S[(size_t)k * D + col] : 0.f;
    }
  } else {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) st[i] = 0.f;
  }
  if (tid < D) {
    r_s[tid] = in[tid];
    k_s[tid] = in[p.off + tid];
    const float* low = p.low + (size_t)b * p.low_stride;
    float acc = p.w0[hc + tid];
    auto add = [&](const uint4& u, int i) {  // the row's padding is zero: elements beyond the rank only need to be finite
      const float4 x = ld4_masked(low, 8 * i, p.rank), y = ld4_masked(low, 8 * i + 4, p.rank);
      acc = fmaf(bf_lo(u.x), x.x, acc); acc = fmaf(bf_hi(u.x), x.y, acc); acc = fmaf(bf_lo(u.y), x.z, acc); acc = fmaf(bf_hi(u.y), x.w, acc);
      acc = fmaf(bf_lo(u.z), y.x, acc); acc = fmaf(bf_hi(u.z), y.y, acc); acc = fmaf(bf_lo(u.w), y.z, acc); acc = fmaf(bf_hi(u.w), y.w, acc);
    };
#pragma unroll
    for (int i = 0; i < W2_KEEP; ++i)
      if (i < rp) add(wk[i], i);
    for (int i = W2_KEEP; i < rp; ++i) add(ldg128(w2 + i), i);
    w_s[tid] = expf(-expf(acc));
  }
  __syncthreads();
  float o = 0.f;
  if (active) {
    const float v = in[2 * p.off + col];
    auto one = [&](int k, float s) -> float {
      const float kv = k_s[k] * v;
      o = fmaf(r_s[k], fmaf(p.u[hc + k], kv, s), o);
      return fmaf(w_s[k], s, kv);
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int k = grp + i * groups;
      if (k < D) S[(size_t)k * D + col] = one(k, st[i]);
    }
    for (int k = grp + KEEP * groups; k < D; k += groups) S[(size_t)k * D + col] = one(k, pos > 0 ? S[(size_t)k * D + col] : 0.f);
    part[grp * D + col] = o;
  }
  __syncthreads();
  float tot = 0.f;
  if (tid < D)
    for (int g = 0; g < groups; ++g) tot += part[g * D + tid];
  float ss[1] = {tot * tot};
  block_sums<1, WKV_STEP_THREADS / 32>(ss, red);
  if (tid < D)
    static_cast<A*>(p.out)[(size_t)b * p.out_stride + hc + tid] =
        to_operand<A>(tot * (1.0f / sqrtf(ss[0] / (float)D + p.eps)) * p.norm[hc + tid] * in[3 * p.off + tid]);
}

constexpr int WKV_SCAN_THREADS = 128;
constexpr int WKV_TILE = 16;  // tokens staged per step
constexpr int WKV_NC = 2;     // value columns per thread

// two FP32 numbers in one 64-bit register pair; each half of an operation rounds like its scalar form
typedef unsigned long long F2;
__device__ __forceinline__ F2 f2(float lo, float hi) {
  F2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float f2_lo(F2 v) { return __uint_as_float((uint32_t)v); }
__device__ __forceinline__ float f2_hi(F2 v) { return __uint_as_float((uint32_t)(v >> 32)); }
__device__ __forceinline__ F2 fma2(F2 a, F2 b, F2 c) {
  F2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ F2 mul2(F2 a, F2 b) {
  F2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

struct WkvScanParams {
  const float* rkv;    // [T][stride]: r, k, v at offsets 0, off, 2 off
  int stride, off;
  const float* decay;  // [T][decay_stride]
  int decay_stride;
  const float* u;      // [heads * dim]
  float* state;        // [slot][heads][dim][dim]
  const RunDesc* runs;
  int heads, dim;
  float* o;            // [T][o_stride]
  int o_stride;
  // the row the next run's token shift starts from: h of the run's last token
  const float* h;
  int h_stride, W;
  float* shift;        // [slot][2][shift_stride]
  int shift_stride;
};

// keys per thread, and lanes per value column: a power of two up to 32 with lanes * keys >= dim
__host__ __device__ __forceinline__ int wkv_keys(int dim) { return dim <= 128 ? 4 : 8; }
__host__ __device__ __forceinline__ int wkv_lanes(int dim) {
  int l = 1;
  while (l * wkv_keys(dim) < dim) l *= 2;
  return l;
}
__host__ __device__ __forceinline__ int wkv_cols(int dim) { return WKV_NC * WKV_SCAN_THREADS / wkv_lanes(dim); }
// tiles in flight: four, or two where a token's row is long
__host__ __device__ constexpr int wkv_stages(int row_keys) { return row_keys <= 128 ? 4 : 2; }
__host__ __device__ __forceinline__ size_t wkv_scan_smem(int dim) {
  return (size_t)wkv_stages(wkv_lanes(dim) * wkv_keys(dim)) * WKV_TILE * (3 * wkv_lanes(dim) * wkv_keys(dim) + wkv_cols(dim)) * 4;
}

// grid = (column blocks of a head, heads, runs). L = lanes per column, KPT = keys per thread; a thread has two columns, COLS / 2 apart.
template <int L, int KPT>
__global__ void __launch_bounds__(WKV_SCAN_THREADS) wkv_scan_kernel(const WkvScanParams p) {
  extern __shared__ __align__(16) float scan_s[];  // ring of tiles of [token][r | k | w (DP each) | v (COLS)]
  constexpr int DP = L * KPT, HALF = WKV_SCAN_THREADS / L, COLS = WKV_NC * HALF, ROW = 3 * DP + COLS;
  constexpr int G = L < WKV_TILE ? L : WKV_TILE;   // tokens whose outputs are reduced together
  constexpr int STAGES = wkv_stages(DP);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, D = p.dim, hc = h * D;
  const RunDesc run = p.runs[blockIdx.z];
  const int ln = tid % L, cl = tid / L, c0 = blockIdx.x * COLS;  // columns c0 + cl and c0 + cl + HALF
  auto key = [&](int i) { return ln * 4 + (i & 3) + (i >> 2) * (DP / 2); };  // runs of four keys: neighbouring lanes read neighbouring 16 bytes
  float* S = p.state + ((size_t)run.slot * p.heads + h) * D * D;
  F2 st[WKV_NC][KPT / 2], u[KPT / 2];  // pairs of neighbouring keys: packed FP32 arithmetic
#pragma unroll
  for (int i = 0; i < KPT / 2; ++i) {
    const int k = key(2 * i);
    u[i] = f2(k < D ? p.u[hc + k] : 0.f, k + 1 < D ? p.u[hc + k + 1] : 0.f);
#pragma unroll
    for (int n = 0; n < WKV_NC; ++n) {
      const int col = c0 + cl + n * HALF;
      const bool ok = run.start > 0 && col < D;
      st[n][i] = f2(ok && k < D ? S[(size_t)k * D + col] : 0.f, ok && k + 1 < D ? S[(size_t)(k + 1) * D + col] : 0.f);
    }
  }
  // padding keys and columns stay zero in every tile of the ring
  for (int i = tid; i < STAGES * WKV_TILE * ROW; i += WKV_SCAN_THREADS) scan_s[i] = 0.f;
  __syncthreads();
  const bool vec = !((D | hc | p.stride | p.off | p.decay_stride) & 3);  // 16-byte pieces possible
  const int nv = min(COLS, D - c0);
  auto cp4 = [](float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
  };
  auto fetch = [&](int tile) {  // a warp takes every fourth token of the tile
    const int first = tile * WKV_TILE, n = min(WKV_TILE, run.len - first);
    for (int t = warp; t < n; t += WKV_SCAN_THREADS / 32) {
      float* d = scan_s + (size_t)((tile % STAGES) * WKV_TILE + t) * ROW;
      const size_t row = (size_t)(run.row0 + first + t);
      const float* rk = p.rkv + row * p.stride + hc;
      const float* dec = p.decay + row * p.decay_stride + hc;
      if (vec) {
        for (int c = lane * 4; c < D; c += 128) {
          pfa_cp16(d + c, rk + c);
          pfa_cp16(d + DP + c, rk + p.off + c);
          pfa_cp16(d + 2 * DP + c, dec + c);
        }
      } else {
        for (int c = lane; c < D; c += 32) {
          cp4(d + c, rk + c);
          cp4(d + DP + c, rk + p.off + c);
          cp4(d + 2 * DP + c, dec + c);
        }
      }
      for (int c = lane; c < nv; c += 32) cp4(d + 3 * DP + c, rk + 2 * p.off + c0 + c);
    }
  };
  const int tiles = (run.len + WKV_TILE - 1) / WKV_TILE;
  auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };
  for (int i = 0; i < STAGES - 1; ++i) {  // one group per tile, empty ones beyond the last
    if (i < tiles) fetch(i);
    commit();
  }
  for (int tile = 0; tile < tiles; ++tile) {
    asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
    __syncthreads();  // the tile has landed for everyone, and everyone has left the one that is refilled now
    if (tile + STAGES - 1 < tiles) fetch(tile + STAGES - 1);
    commit();
    const float* base = scan_s + (size_t)(tile % STAGES) * WKV_TILE * ROW;
    const int n = min(WKV_TILE, run.len - tile * WKV_TILE);
    auto group = [&](int g0, auto whole) {  // tokens g0 .. g0 + G - 1 of the tile
      float o[WKV_NC][G];
#pragma unroll
      for (int j = 0; j < G; ++j) {
#pragma unroll
        for (int c = 0; c < WKV_NC; ++c) o[c][j] = 0.f;
        if (!decltype(whole)::value && g0 + j >= n) continue;
        const float* row = base + (g0 + j) * ROW;
        auto pairs = [&](const float* src, F2 (&v)[KPT / 2]) {
#pragma unroll
          for (int i = 0; i < KPT / 4; ++i) {
            const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(src + i * (DP / 2) + ln * 4);
            v[2 * i] = a.x; v[2 * i + 1] = a.y;
          }
        };
        F2 r[KPT / 2], k[KPT / 2], w[KPT / 2];
        pairs(row, r);
        pairs(row + DP, k);
        pairs(row + 2 * DP, w);
#pragma unroll
        for (int c = 0; c < WKV_NC; ++c) {
          const float v1 = row[3 * DP + cl + c * HALF];
          const F2 v = f2(v1, v1);
          F2 acc = f2(0.f, 0.f);
#pragma unroll
          for (int i = 0; i < KPT / 2; ++i) {
            const F2 kv = mul2(k[i], v);
            acc = fma2(r[i], fma2(u[i], kv, st[c][i]), acc);
            st[c][i] = fma2(w[i], st[c][i], kv);
          }
          o[c][j] = f2_lo(acc) + f2_hi(acc);
        }
      }
      // sums over the column's lanes; lane j (mod G) ends up with token j
#pragma unroll
      for (int c = 0; c < WKV_NC; ++c) {
        if (L > G)
#pragma unroll
          for (int j = 0; j < G; ++j) o[c][j] += __shfl_xor_sync(0xffffffffu, o[c][j], L / 2);
#pragma unroll
        for (int s = G / 2; s > 0; s >>= 1)
#pragma unroll
          for (int j = 0; j < s; ++j) {
            const bool up = ln & s;
            const float send = up ? o[c][j] : o[c][j + s], keep = up ? o[c][j + s] : o[c][j];
            o[c][j] = keep + __shfl_xor_sync(0xffffffffu, send, s);
          }
        const int t = g0 + ln % G, col = c0 + cl + c * HALF;
        if (ln < G && t < n && col < D) p.o[(size_t)(run.row0 + tile * WKV_TILE + t) * p.o_stride + hc + col] = o[c][0];
      }
    };
    if (n == WKV_TILE)
      for (int g0 = 0; g0 < WKV_TILE; g0 += G) group(g0, std::true_type{});
    else
      for (int g0 = 0; g0 < n; g0 += G) group(g0, std::false_type{});
  }
#pragma unroll
  for (int n = 0; n < WKV_NC; ++n) {
    const int col = c0 + cl + n * HALF;
    if (col < D)
#pragma unroll
      for (int i = 0; i < KPT / 2; ++i) {
        const int k = key(2 * i);
        if (k < D) S[(size_t)k * D + col] = f2_lo(st[n][i]);
        if (k + 1 < D) S[(size_t)(k + 1) * D + col] = f2_hi(st[n][i]);
      }
  }
  if (blockIdx.x == 0) {  // the heads' first blocks share the copy of the last token's h
    const float* src = p.h + (size_t)(run.row0 + run.len - 1) * p.h_stride;
    float* dst = p.shift + ((size_t)run.slot * 2 + ((run.start + run.len) & 1)) * p.shift_stride;
    for (int i = h * WKV_SCAN_THREADS + tid; i < p.W; i += p.heads * WKV_SCAN_THREADS) dst[i] = src[i];
  }
}

}  // namespace b200
