// Latent attention: keys and values of all heads are linear images of one small vector c per token (kv_rank elements,
// RMS-normed), plus one rotated key part of rot_dim elements shared by the heads. The cache holds only [c | rotated
// part] per token, in rows padded to multiples of 8 elements; a sliding window keeps the cache a ring of `cap` rows
// (position p in row p % cap), cap >= window - 1 + tokens per launch.
//
//   latent_append_kernel   prompts: norm + rotation of new rows into the ring, and the rows a chunk attends to laid out
//                          contiguously (history from the ring, then the new ones) for the key / value expansion
//   latent_prefill_kernel  prompts: 64 queries of one head per block over expanded keys and values, 64-key tiles, online
//                          softmax, bfloat16 tensor-core products (mma.sync m16n8k16) with FP32 scores and sums
//   latent_decode_kernel   one token of several sequences: works on the latents themselves. The query's unrotated part is
//                          taken through W_uk once (q . W_uk c = (W_uk^T q) . c), scores and the weighted sum run over c,
//                          and the sum is taken through W_uv at the end. FP32 arithmetic on the cached rows.
//
// A = type of the cache and of matmul operands: __nv_bfloat16, or float in a 32-bit engine.
#pragma once
#include "attn_prefill.cuh"
#include "block_rows.cuh"

namespace b200 {

__device__ __forceinline__ float from_operand(float v) { return v; }
__device__ __forceinline__ float from_operand(__nv_bfloat16 v) { return __bfloat162float(v); }
// eight consecutive elements (16- or 32-byte aligned)
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  v[0] = bf_lo(u.x); v[1] = bf_hi(u.x); v[2] = bf_lo(u.y); v[3] = bf_hi(u.y);
  v[4] = bf_lo(u.z); v[5] = bf_hi(u.z); v[6] = bf_lo(u.w); v[7] = bf_hi(u.w);
}
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}

// Element i of a rotated vector: pairs (2j, 2j+1) for j < pairs, table row = {cos, sin} per pair; the rest passes.
__device__ __forceinline__ float rotated(const float* v, int i, const float* rope_row, int pairs) {
  const int j = i >> 1;
  if (j >= pairs) return v[i];
  const float c = rope_row[2 * j], s = rope_row[2 * j + 1];
  return (i & 1) ? v[i] * c + v[i - 1] * s : v[i] * c - v[i + 1] * s;
}

struct LatentAppendParams {
  const float* low;    // [T][low_stride]: raw W_dkv h (kv_rank, then rot_dim)
  int low_stride, kv_rank, rot_dim;
  const float* c_norm;
  float eps;
  const float* rope;   // [max_ctx][pairs]{cos, sin}
  int pairs;
  void* cache;         // [slot][cap][crow]
  int crow, kvp, cap;  // kvp = pad8(kv_rank), crow = kvp + pad8(rot_dim)
  const RunDesc* runs;
  int nruns, rows;     // rows = context rows of all runs
  void* ctx;           // [rows][kvp] latents, or nullptr (no expansion: `rows` counts new rows only)
  void* kr;            // [rows][crow - kvp] rotated parts
};

// One warp per context row.
template <typename A>
__global__ void __launch_bounds__(256) latent_append_kernel(const LatentAppendParams p) {
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= p.rows) return;
  int lo = 0, hi = p.nruns - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.runs[mid].ctx0 <= row) lo = mid;
    else hi = mid - 1;
  }
  const RunDesc r = p.runs[lo];
  const int idx = row - r.ctx0, pos = r.start - r.hist + idx, rp = p.crow - p.kvp;
  A* cache = static_cast<A*>(p.cache) + ((size_t)r.slot * p.cap + pos % p.cap) * p.crow;
  A* ctx = p.ctx ? static_cast<A*>(p.ctx) + (size_t)row * p.kvp : nullptr;
  A* kr = p.ctx ? static_cast<A*>(p.kr) + (size_t)row * rp : nullptr;
  if (idx < r.hist) {
    for (int i = lane; i < p.kvp; i += 32) ctx[i] = cache[i];
    for (int i = lane; i < rp; i += 32) kr[i] = cache[p.kvp + i];
    return;
  }
  const float* in = p.low + (size_t)(r.row0 + idx - r.hist) * p.low_stride;
  float ss = 0.f;
  for (int i = lane; i < p.kv_rank; i += 32) ss += in[i] * in[i];
  const float f = 1.0f / sqrtf(warp_sum(ss) / (float)p.kv_rank + p.eps);
  for (int i = lane; i < p.kv_rank; i += 32) {
    const A v = to_operand<A>(in[i] * f * p.c_norm[i]);
    cache[i] = v;
    if (ctx) ctx[i] = v;
  }
  const float* table = p.rope + (size_t)pos * p.pairs * 2;
  for (int i = lane; i < p.rot_dim; i += 32) {
    const A v = to_operand<A>(rotated(in + p.kv_rank, i, table, p.pairs));
    cache[p.kvp + i] = v;
    if (kr) kr[i] = v;
  }
}

// ---- decode ------------------------------------------------------------------------------------------------------
constexpr int LAD_THREADS = 256, LAD_WARPS = LAD_THREADS / 32;
constexpr int LAD_MAX_SPLITS = 64;

struct LatentDecodeParams {
  const float* q;       // [batch][q_stride]: per head dim unrotated, then rot_dim (rotated here)
  int q_stride;
  const float* low;     // [batch][low_stride]: raw W_dkv h of the new token
  int low_stride;
  const float* c_norm;
  float eps;
  const float* rope;
  int pairs;
  void* cache;          // [slot][cap][crow]
  int crow, kvp, cap;
  const int* positions;
  const int* slots;
  const __nv_bfloat16* uk;  // [heads * dim][kvp]
  const __nv_bfloat16* uv;  // [heads * vdim][kvp]
  const float* gate;    // [batch][gate_stride]
  int gate_stride;
  int heads, dim, rot_dim, vdim, kv_rank, window, max_ctx;
  float scale;
  int nsplit, split_cap;  // context splits per (head, sequence); most keys of one split
  float* part_o;        // [batch][heads][nsplit][kvp]
  float* part_ml;       // [batch][heads][nsplit][2]
  int* tickets;         // [batch][heads], zero between launches
  void* out;            // [batch][out_stride]: FP32 rows, or matmul operands when out_bf16 is set
  int out_stride, out_bf16;
  int cached_new;       // 1: the new rows are already in the cache
  int* error_flag;
};

// qv (crow) | new row (crow) | o (kvp) | partial sums (LAD_THREADS * 8) | unrotated query (dim) | scores (split_cap)
__host__ __device__ __forceinline__ size_t lad_smem_bytes(int crow, int kvp, int dim, int split_cap) {
  return (size_t)(2 * crow + kvp + LAD_THREADS * 8 + pad8(dim) + split_cap) * 4;
}

// Column sums of a weighted set of rows: out[j] = sum_i weight(i) * row(i)[j] for j < ncol (a multiple of 8). A thread
// owns eight columns; `groups` sets of threads take every groups-th row and are added up in order through `part`.
template <typename Row, typename Weight>
__device__ __forceinline__ void weighted_rows(int n, int ncol, Row row, Weight weight, float* part, float* out) {
  const int tid = threadIdx.x, nch = ncol >> 3;
  const int span = min(nch, LAD_THREADS), groups = LAD_THREADS / span;
  const int grp = tid / span, ch = tid - grp * span;
  for (int c0 = 0; c0 < nch; c0 += span) {
    const int c = c0 + ch;
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (grp < groups && c < nch) {
#pragma unroll 8
      for (int i = grp; i < n; i += groups) {
        float v[8];
        load8(row(i) + 8 * c, v);
        const float w = weight(i);
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = fmaf(w, v[e], acc[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) part[e * LAD_THREADS + tid] = acc[e];
    __syncthreads();
    for (int i = tid; i < 8 * span; i += LAD_THREADS) {
      const int e = i / span, cc = i - e * span;
      if (c0 + cc < nch) {
        float t = 0.f;
        for (int g = 0; g < groups; ++g) t += part[e * LAD_THREADS + g * span + cc];
        out[8 * (c0 + cc) + e] = t;
      }
    }
    __syncthreads();
  }
}

// grid = (splits, heads, batch). A = cache type, O = type of the output rows.
template <typename A, typename O>
__global__ void __launch_bounds__(LAD_THREADS) latent_decode_kernel(const LatentDecodeParams p) {
  extern __shared__ __align__(16) float lad_s[];
  __shared__ float red[LAD_WARPS], ml_s[2 * LAD_MAX_SPLITS];
  __shared__ int last_s;
  float* qv = lad_s;                          // query in the layout of a cache row, scaled
  float* nr = qv + p.crow;                    // the new token's cache row
  float* ol = nr + p.crow;                    // weighted sum of latents
  float* part = ol + p.kvp;
  float* qn = part + LAD_THREADS * 8;
  float* sc = qn + pad8(p.dim);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int split = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  pdl_launch_dependents();
  const __nv_bfloat16* uk = p.uk + (size_t)h * p.dim * p.kvp;
  const __nv_bfloat16* uv = p.uv + (size_t)h * p.vdim * p.kvp;
  {  // this head's weights into L2 while the previous kernel still runs: they depend on nothing
    const size_t nk = (size_t)p.dim * p.kvp * 2, nv = (size_t)p.vdim * p.kvp * 2;
    for (size_t o = (size_t)(split * LAD_THREADS + tid) * 128; o < nk; o += (size_t)p.nsplit * LAD_THREADS * 128)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(uk) + o));
    for (size_t o = (size_t)(split * LAD_THREADS + tid) * 128; o < nv; o += (size_t)p.nsplit * LAD_THREADS * 128)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(uv) + o));
  }
  pdl_wait();
  const int pos = p.positions[b], slot = p.slots[b];
  if (pos < 0 || pos >= p.max_ctx) {  // nothing is read or appended for this sequence
    if (tid == 0 && p.error_flag) *reinterpret_cast<volatile int*>(p.error_flag) = 3;
    return;
  }
  A* cache = static_cast<A*>(p.cache) + (size_t)slot * p.cap * p.crow;
  const float* table = p.rope + (size_t)pos * p.pairs * 2;
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0, nkeys = pos - lo + 1;
  const int chunk = (nkeys + p.nsplit - 1) / p.nsplit;
  const int t0 = lo + split * chunk, t1 = min(pos + 1, t0 + chunk), n = max(0, t1 - t0);

  // ---- the new token's row, and the query ----
  const float* qh = p.q + (size_t)b * p.q_stride + h * (p.dim + p.rot_dim);
  for (int i = tid; i < p.dim; i += LAD_THREADS) qn[i] = qh[i];
  for (int i = tid; i < p.crow - p.kvp; i += LAD_THREADS) qv[p.kvp + i] = i < p.rot_dim ? rotated(qh + p.dim, i, table, p.pairs) * p.scale : 0.f;
  if (!p.cached_new) {
    const float* in = p.low + (size_t)b * p.low_stride;
    float ss[1] = {0.f};
    for (int i = tid; i < p.kv_rank; i += LAD_THREADS) ss[0] += in[i] * in[i];
    block_sums<1, LAD_WARPS>(ss, red);
    const float f = 1.0f / sqrtf(ss[0] / (float)p.kv_rank + p.eps);
    const bool owner = h == 0 && pos >= t0 && pos < t1;
    A* row = cache + (size_t)(pos % p.cap) * p.crow;
    for (int i = tid; i < p.crow; i += LAD_THREADS) {
      float v = 0.f;
      if (i < p.kv_rank) v = in[i] * f * p.c_norm[i];
      else if (i >= p.kvp && i - p.kvp < p.rot_dim) v = rotated(in + p.kv_rank, i - p.kvp, table, p.pairs);
      const A a = to_operand<A>(v);
      nr[i] = from_operand(a);
      if (owner) row[i] = a;
    }
  }
  __syncthreads();
  // ---- query through W_uk^T ----
  weighted_rows(p.dim, p.kvp, [&](int d) { return uk + (size_t)d * p.kvp; }, [&](int d) { return qn[d] * p.scale; }, part, qv);

  // ---- scores: a warp takes four keys at a time ----
  const bool from_smem = !p.cached_new;
  const int nch = p.crow >> 3;
  float mx = -INFINITY;
  for (int k0 = warp * 4; k0 < n; k0 += LAD_WARPS * 4) {
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    const A* rows[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) rows[e] = cache + (size_t)((t0 + min(k0 + e, n - 1)) % p.cap) * p.crow;
    for (int c = lane; c < nch; c += 32) {
      float qc[8];
      load8(qv + 8 * c, qc);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float kv[8];
        load8(rows[e] + 8 * c, kv);
#pragma unroll
        for (int i = 0; i < 8; ++i) s[e] = fmaf(qc[i], kv[i], s[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      s[e] = warp_sum(s[e]);
      if (from_smem && t0 + k0 + e == pos) {  // the newest row is not in the cache yet for everyone
        float v = 0.f;
        for (int i = lane; i < p.crow; i += 32) v = fmaf(qv[i], nr[i], v);
        s[e] = warp_sum(v);
      }
      if (k0 + e < n) mx = fmaxf(mx, s[e]);
    }
    if (lane < 4 && k0 + lane < n) sc[k0 + lane] = lane == 0 ? s[0] : lane == 1 ? s[1] : lane == 2 ? s[2] : s[3];
  }
  if (lane == 0) red[warp] = mx;
  __syncthreads();
  mx = red[0];
#pragma unroll
  for (int w = 1; w < LAD_WARPS; ++w) mx = fmaxf(mx, red[w]);
  __syncthreads();
  float sum[1] = {0.f};
  for (int k = tid; k < n; k += LAD_THREADS) {
    const float e = expf(sc[k] - mx);
    sc[k] = e;
    sum[0] += e;
  }
  block_sums<1, LAD_WARPS>(sum, red);

  // ---- weighted sum of the latents ----
  const int own = from_smem && pos >= t0 && pos < t1 ? pos - t0 : -1;
  weighted_rows(own >= 0 ? n - 1 : n, p.kvp, [&](int k) { return cache + (size_t)((t0 + k) % p.cap) * p.crow; }, [&](int k) { return sc[k]; }, part, ol);
  if (own >= 0) {
    for (int i = tid; i < p.kvp; i += LAD_THREADS) ol[i] = fmaf(sc[own], nr[i], ol[i]);
    __syncthreads();
  }
  float total = sum[0];
  if (p.nsplit > 1) {
    const size_t base = ((size_t)b * p.heads + h) * p.nsplit;
    for (int i = tid; i < p.kvp; i += LAD_THREADS) p.part_o[(base + split) * p.kvp + i] = ol[i];
    if (tid == 0) {
      p.part_ml[(base + split) * 2] = mx;
      p.part_ml[(base + split) * 2 + 1] = total;
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) last_s = atomicAdd(&p.tickets[(size_t)b * p.heads + h], 1) == p.nsplit - 1;
    __syncthreads();
    if (!last_s) return;
    __threadfence();
    if (tid == 0) p.tickets[(size_t)b * p.heads + h] = 0;
    if (tid < 2 * p.nsplit) ml_s[tid] = __ldcg(&p.part_ml[base * 2 + tid]);
    __syncthreads();
    float M = -INFINITY;
    for (int s = 0; s < p.nsplit; ++s)
      if (ml_s[2 * s + 1] > 0.f) M = fmaxf(M, ml_s[2 * s]);
    total = 0.f;
    for (int s = 0; s < p.nsplit; ++s)
      if (ml_s[2 * s + 1] > 0.f) total += ml_s[2 * s + 1] * expf(ml_s[2 * s] - M);
    for (int i = tid; i < p.kvp; i += LAD_THREADS) {
      float o = 0.f;
#pragma unroll 8
      for (int s = 0; s < p.nsplit; ++s) {
        const float v = __ldcg(&p.part_o[(base + s) * p.kvp + i]);
        if (ml_s[2 * s + 1] > 0.f) o = fmaf(expf(ml_s[2 * s] - M), v, o);
      }
      ol[i] = o;
    }
    __syncthreads();
  }
  // ---- through W_uv, times the gate ----
  const float inv = 1.0f / total;
  const int vch = p.kvp >> 3;
  for (int r0 = warp * 4; r0 < p.vdim; r0 += LAD_WARPS * 4) {
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    for (int c = lane; c < vch; c += 32) {
      float oc[8];
      load8(ol + 8 * c, oc);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float w[8];
        load8(uv + (size_t)min(r0 + e, p.vdim - 1) * p.kvp + 8 * c, w);
#pragma unroll
        for (int i = 0; i < 8; ++i) s[e] = fmaf(w[i], oc[i], s[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) s[e] = warp_sum(s[e]);
    if (lane < 4 && r0 + lane < p.vdim) {
      const float v = (lane == 0 ? s[0] : lane == 1 ? s[1] : lane == 2 ? s[2] : s[3]) * inv;
      const int j = h * p.vdim + r0 + lane;
      static_cast<O*>(p.out)[(size_t)b * p.out_stride + j] = to_operand<O>(v * p.gate[(size_t)b * p.gate_stride + j]);
    }
  }
}

// ---- prompts -----------------------------------------------------------------------------------------------------
constexpr int LAP_Q = 64, LAP_K = 64, LAP_THREADS = 128;

struct LatentPrefillParams {
  const float* q;            // [T][q_stride], unrotated
  int q_stride;
  const float* rope;
  int pairs;
  const __nv_bfloat16* kv;   // [context rows][kv_stride]: unrotated keys of all heads, values from column v_off on
  int kv_stride, v_off;
  const __nv_bfloat16* kr;   // [context rows][kr_stride] rotated key parts
  int kr_stride;
  const float* gate;         // [T][gate_stride]
  int gate_stride;
  const RunDesc* runs;
  int heads, dim, rot_dim, vdim, window;
  float scale;
  __nv_bfloat16* out;        // [T][out_stride]
  int out_stride;
};

__host__ __device__ __forceinline__ int lap_qk_stride(int dim, int rot) { return (dim + rot + 15) / 16 * 16 + 8; }
__host__ __device__ __forceinline__ size_t lap_smem_bytes(int dim, int rot, int vp) {
  return ((size_t)(LAP_Q + LAP_K) * lap_qk_stride(dim, rot) + (size_t)LAP_K * (vp + 8)) * 2;
}

__device__ __forceinline__ void lap_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf2(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}

// grid = (query blocks of the longest run, heads, runs). VP = value columns per head rounded up to 32, 64, 128 or 256.
template <int VP>
__global__ void __launch_bounds__(LAP_THREADS) latent_prefill_kernel(const LatentPrefillParams p) {
  extern __shared__ __align__(16) unsigned char lap_smem[];
  const RunDesc run = p.runs[blockIdx.z];
  const int q0 = blockIdx.x * LAP_Q, h = blockIdx.y;
  if (q0 >= run.len) return;
  const int E = p.dim + p.rot_dim, EP = (E + 15) / 16 * 16, QS = EP + 8;
  constexpr int VS = VP + 8, NT_O = VP / 8;
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(lap_smem);
  __nv_bfloat16* Ks = Qs + LAP_Q * QS;
  __nv_bfloat16* Vs = Ks + LAP_K * QS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int nq = min(LAP_Q, run.len - q0);
  // queries: rotated, scaled into the base-2 exponent domain only after the product
  for (int i = tid; i < LAP_Q * EP; i += LAP_THREADS) {
    const int r = i / EP, c = i - r * EP;
    float v = 0.f;
    if (r < nq && c < E) {
      const float* qr = p.q + (size_t)(run.row0 + q0 + r) * p.q_stride + h * E;
      v = c < p.dim ? qr[c] : rotated(qr + p.dim, c - p.dim, p.rope + (size_t)(run.start + q0 + r) * p.pairs * 2, p.pairs);
    }
    Qs[r * QS + c] = __float2bfloat16(v);
  }
  const int qpos0 = run.start + q0;                       // position of the block's first query
  const int kfirst = p.window > 0 ? max(0, qpos0 - p.window + 1) : 0, klast = qpos0 + nq - 1;
  const int base = run.start - run.hist;                  // position of the run's first context row
  const int my0 = qpos0 + warp * 16 + g, my1 = my0 + 8;   // this thread's two query positions
  const int win = p.window > 0 ? p.window : 0x7fffffff;
  float o[NT_O][4];
#pragma unroll
  for (int i = 0; i < NT_O; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  const float sc2 = p.scale * 1.4426950408889634f;
  const bool vec = !((p.dim | p.rot_dim | p.vdim | p.kv_stride | p.v_off | p.kr_stride) & 7);

  for (int kt = kfirst; kt <= klast; kt += LAP_K) {
    const int nk = min(LAP_K, klast - kt + 1);
    __syncthreads();  // the previous tile (or the query tile's writers) are done
    const size_t crow = (size_t)(run.ctx0 + kt - base);
    if (vec) {
      const int ce = EP >> 3, cd = p.dim >> 3, cn = E >> 3, cv = VP >> 3, cvn = p.vdim >> 3;
      for (int i = tid; i < LAP_K * ce; i += LAP_THREADS) {
        const int r = i / ce, c = i - r * ce;
        __nv_bfloat16* d = Ks + r * QS + 8 * c;
        if (r < nk && c < cn)
          pfa_cp16(d, c < cd ? p.kv + (crow + r) * p.kv_stride + h * p.dim + 8 * c : p.kr + (crow + r) * p.kr_stride + 8 * (c - cd));
        else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
      }
      for (int i = tid; i < LAP_K * cv; i += LAP_THREADS) {
        const int r = i / cv, c = i - r * cv;
        __nv_bfloat16* d = Vs + r * VS + 8 * c;
        if (r < nk && c < cvn) pfa_cp16(d, p.kv + (crow + r) * p.kv_stride + p.v_off + h * p.vdim + 8 * c);
        else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
      }
      pfa_cp_wait_all();
    } else {
      const __nv_bfloat16 zero = __float2bfloat16(0.f);
      for (int i = tid; i < LAP_K * EP; i += LAP_THREADS) {
        const int r = i / EP, c = i - r * EP;
        __nv_bfloat16 v = zero;
        if (r < nk && c < E) v = c < p.dim ? p.kv[(crow + r) * p.kv_stride + h * p.dim + c] : p.kr[(crow + r) * p.kr_stride + c - p.dim];
        Ks[r * QS + c] = v;
      }
      for (int i = tid; i < LAP_K * VP; i += LAP_THREADS) {
        const int r = i / VP, c = i - r * VP;
        Vs[r * VS + c] = r < nk && c < p.vdim ? p.kv[(crow + r) * p.kv_stride + p.v_off + h * p.vdim + c] : zero;
      }
    }
    __syncthreads();
    // scores: 16 queries x 64 keys per warp
    float s[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    for (int ks = 0; ks < EP; ks += 16) {
      uint32_t a[4];
      pfa_ldm4(a, Qs + (warp * 16 + (lane & 15)) * QS + ks + (lane >> 4) * 8);
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {  // 16 keys: two 8-key fragments
        uint32_t kb[4];
        pfa_ldm4(kb, Ks + (nt * 16 + (lane & 7) + (lane >> 4) * 8) * QS + ks + ((lane >> 3) & 1) * 8);
        lap_mma(s[2 * nt], a, kb[0], kb[1]);
        lap_mma(s[2 * nt + 1], a, kb[2], kb[3]);
      }
    }
    float n0 = m0, n1 = m1;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int key = kt + 8 * i + 2 * t + e;
        s[i][e] = key <= my0 && my0 - key < win ? s[i][e] * sc2 : -INFINITY;
        s[i][2 + e] = key <= my1 && my1 - key < win ? s[i][2 + e] * sc2 : -INFINITY;
        n0 = fmaxf(n0, s[i][e]);
        n1 = fmaxf(n1, s[i][2 + e]);
      }
    }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
      n0 = fmaxf(n0, __shfl_xor_sync(0xffffffffu, n0, x));
      n1 = fmaxf(n1, __shfl_xor_sync(0xffffffffu, n1, x));
    }
    // a row that has seen no key yet keeps -infinity: subtract 0 then, every weight is exp2(-inf) = 0
    const float z0 = n0 == -INFINITY ? 0.f : n0, z1 = n1 == -INFINITY ? 0.f : n1;
    const float f0 = exp2f(m0 - z0), f1 = exp2f(m1 - z1);
    m0 = n0; m1 = n1;
    l0 *= f0; l1 *= f1;
#pragma unroll
    for (int i = 0; i < NT_O; ++i) { o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1; }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        s[i][e] = exp2f(s[i][e] - z0);
        s[i][2 + e] = exp2f(s[i][2 + e] - z1);
        l0 += s[i][e];
        l1 += s[i][2 + e];
      }
    }
    // weighted values
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      const uint32_t a[4] = {pack_bf2(s[2 * kk][0], s[2 * kk][1]), pack_bf2(s[2 * kk][2], s[2 * kk][3]), pack_bf2(s[2 * kk + 1][0], s[2 * kk + 1][1]),
                             pack_bf2(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
      for (int nt = 0; nt < NT_O / 2; ++nt) {
        uint32_t vb[4];
        pfa_ldm4t(vb, Vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VS + nt * 16 + (lane >> 4) * 8);
        lap_mma(o[2 * nt], a, vb[0], vb[1]);
        lap_mma(o[2 * nt + 1], a, vb[2], vb[3]);
      }
    }
  }
#pragma unroll
  for (int x = 1; x < 4; x <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, x);
    l1 += __shfl_xor_sync(0xffffffffu, l1, x);
  }
  const float i0 = 1.0f / l0, i1 = 1.0f / l1;
#pragma unroll
  for (int i = 0; i < NT_O; ++i) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = warp * 16 + g + (e >> 1) * 8, c = 8 * i + 2 * t + (e & 1);
      if (r < nq && c < p.vdim) {
        const size_t row = (size_t)(run.row0 + q0 + r);
        const int j = h * p.vdim + c;
        p.out[row * p.out_stride + j] = __float2bfloat16(o[i][e] * (e < 2 ? i0 : i1) * p.gate[row * p.gate_stride + j]);
      }
    }
  }
}

}  // namespace b200
