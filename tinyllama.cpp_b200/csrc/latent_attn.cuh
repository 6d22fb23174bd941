// Latent attention: keys and values of all heads are linear images of one small vector c per token (kv_rank elements,
// RMS-normed), plus one rotated key part of rot_dim elements shared by the heads. The cache holds only [c | rotated
// part] per token, in rows padded to multiples of 8 elements; a sliding window keeps the cache a ring of `cap` rows
// (position p in row p % cap), cap >= window - 1 + tokens per launch.
//
//   latent_append_kernel   prompts: norm + rotation of new rows into the ring, and the rows a chunk attends to laid out
//                          contiguously (history from the ring, then the new ones) for the key / value expansion
//   latent_prefill_kernel  prompts: 128 queries of one head per block over expanded keys and values, 64-key tiles, online
//                          softmax, bfloat16 tensor-core products (mma.sync m16n8k16) with FP32 scores and sums
//   decode                 one token of several sequences: works on the latents themselves. The query's unrotated part is
//                          taken through W_uk once (q . W_uk c = (W_uk^T q) . c), scores and the weighted sum run over c,
//                          and the sum is taken through W_uv at the end. latent_decode_kernel does all of it for one
//                          head in FP32 (32-bit engines); bfloat16 engines split it into three launches
//                          (latent_absorb_kernel, latent_split_kernel, latent_merge_kernel)
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

// ---- decode on the tensor cores (bfloat16 cache) -------------------------------------------------------------------
// Three launches: latent_absorb_kernel takes the queries through W_uk and appends the new rows, latent_split_kernel runs
// scores and weighted sums for 16 heads and one run of keys per block, latent_merge_kernel merges the runs and goes
// through W_uv. The cached rows are bfloat16 as they are; queries and attention weights enter the products as the sum of
// two bfloat16 numbers (value and remainder), so that they keep 16 bits of mantissa and the scores FP32 character.

__device__ __forceinline__ void split_bf16(float v, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16(v);
  lo = __float2bfloat16(v - __bfloat162float(hi));
}

constexpr int LAB_THREADS = 256;
constexpr int LAB_COLS = 64;   // latent columns per block
constexpr int LAB_BATCH = 8;   // sequences per block
constexpr int LAB_KEEP = 8;    // pieces of W_uk a thread requests ahead (dim up to 256)

struct LatentAbsorbParams {
  LatentDecodeParams d;
  __nv_bfloat16* q_hi;  // [batch][heads][qrow]: scaled query in the layout of a cache row, zero-filled up to qrow
  __nv_bfloat16* q_lo;
  int qrow, batch;
};

// grid = (kvp / 64 rounded up, then one more, heads, batch / 8 rounded up): the last block of a head rotates the queries'
// other part and, for head 0, appends the new cache rows while the others go through W_uk.
__global__ void __launch_bounds__(LAB_THREADS) latent_absorb_kernel(const LatentAbsorbParams a) {
  const LatentDecodeParams& p = a.d;
  extern __shared__ __align__(16) float lab_s[];  // queries [LAB_BATCH][dim], then partial sums [8 warps][LAB_BATCH][64]
  __shared__ float red[LAB_THREADS / 32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y;
  const int b0 = blockIdx.z * LAB_BATCH, nb = min(LAB_BATCH, a.batch - b0);
  float* part = lab_s + LAB_BATCH * p.dim;
  pdl_launch_dependents();
  const int qd = p.dim + p.rot_dim;
  if (blockIdx.x * LAB_COLS >= p.kvp) {
    pdl_wait();
    for (int b = 0; b < nb; ++b) {
      const int pos = p.positions[b0 + b];
      if (pos < 0 || pos >= p.max_ctx) {  // nothing is appended, and the next launch skips the sequence
        if (h == 0 && tid == 0 && p.error_flag) *reinterpret_cast<volatile int*>(p.error_flag) = 3;
        continue;
      }
      const float* table = p.rope + (size_t)pos * p.pairs * 2;
      const float* qr = p.q + (size_t)(b0 + b) * p.q_stride + h * qd + p.dim;
      for (int i = tid; i < a.qrow - p.kvp; i += LAB_THREADS) {
        const size_t at = ((size_t)(b0 + b) * p.heads + h) * a.qrow + p.kvp + i;
        split_bf16(i < p.rot_dim ? rotated(qr, i, table, p.pairs) * p.scale : 0.f, a.q_hi[at], a.q_lo[at]);
      }
      if (h) continue;
      const float* in = p.low + (size_t)(b0 + b) * p.low_stride;
      float ss[1] = {0.f};
      for (int i = tid; i < p.kv_rank; i += LAB_THREADS) ss[0] += in[i] * in[i];
      block_sums<1, LAB_THREADS / 32>(ss, red);
      const float f = 1.0f / sqrtf(ss[0] / (float)p.kv_rank + p.eps);
      __nv_bfloat16* row = static_cast<__nv_bfloat16*>(p.cache) + ((size_t)p.slots[b0 + b] * p.cap + pos % p.cap) * p.crow;
      for (int i = tid; i < p.kv_rank; i += LAB_THREADS) row[i] = __float2bfloat16(in[i] * f * p.c_norm[i]);
      for (int i = tid; i < p.rot_dim; i += LAB_THREADS) row[p.kvp + i] = __float2bfloat16(rotated(in + p.kv_rank, i, table, p.pairs));
    }
    return;
  }
  // thread = (8 columns, every 32nd row of the head's W_uk): pieces requested before anything else
  const int ch = tid & 7, grp = tid >> 3, col = blockIdx.x * LAB_COLS + 8 * ch;
  const bool col_ok = col < p.kvp;
  const __nv_bfloat16* uk = p.uk + (size_t)h * p.dim * p.kvp;
  uint4 w[LAB_KEEP];
#pragma unroll
  for (int i = 0; i < LAB_KEEP; ++i) {
    const int d = grp + 32 * i;
    w[i] = col_ok && d < p.dim ? ldg128(uk + (size_t)d * p.kvp + col) : make_uint4(0, 0, 0, 0);
  }
  pdl_wait();
  for (int i = tid; i < nb * p.dim; i += LAB_THREADS) {
    const int b = i / p.dim, d = i - b * p.dim;
    lab_s[i] = p.q[(size_t)(b0 + b) * p.q_stride + h * qd + d] * p.scale;
  }
  __syncthreads();
  for (int b = 0; b < nb; ++b) {
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    const float* q = lab_s + b * p.dim;
    auto add = [&](const uint4& u, float x) {
      acc[0] = fmaf(bf_lo(u.x), x, acc[0]); acc[1] = fmaf(bf_hi(u.x), x, acc[1]); acc[2] = fmaf(bf_lo(u.y), x, acc[2]); acc[3] = fmaf(bf_hi(u.y), x, acc[3]);
      acc[4] = fmaf(bf_lo(u.z), x, acc[4]); acc[5] = fmaf(bf_hi(u.z), x, acc[5]); acc[6] = fmaf(bf_lo(u.w), x, acc[6]); acc[7] = fmaf(bf_hi(u.w), x, acc[7]);
    };
#pragma unroll
    for (int i = 0; i < LAB_KEEP; ++i)
      if (grp + 32 * i < p.dim) add(w[i], q[grp + 32 * i]);
    for (int d = grp + 32 * LAB_KEEP; d < p.dim; d += 32)
      if (col_ok) add(ldg128(uk + (size_t)d * p.kvp + col), q[d]);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 8);
      acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 16);
    }
    if (lane < 8) {
#pragma unroll
      for (int e = 0; e < 8; ++e) part[(warp * LAB_BATCH + b) * LAB_COLS + 8 * lane + e] = acc[e];
    }
  }
  __syncthreads();
  for (int i = tid; i < nb * LAB_COLS; i += LAB_THREADS) {
    const int b = i / LAB_COLS, c = i - b * LAB_COLS, j = blockIdx.x * LAB_COLS + c;
    if (j >= p.kvp) continue;
    float t = 0.f;
#pragma unroll
    for (int x = 0; x < LAB_THREADS / 32; ++x) t += part[(x * LAB_BATCH + b) * LAB_COLS + c];
    const size_t at = ((size_t)(b0 + b) * p.heads + h) * a.qrow + j;
    split_bf16(t, a.q_hi[at], a.q_lo[at]);
  }
}

constexpr int LAS_THREADS = 256, LAS_WARPS = 8, LAS_HEADS = 16, LAS_KEYS = 64;

__host__ __device__ __forceinline__ int las_row(int n) { return (n + 31) / 32 * 32; }
__host__ __device__ __forceinline__ size_t las_smem_bytes(int crow) {
  const size_t row = las_row(crow) + 8;
  return (LAS_KEYS + 2 * LAS_HEADS) * row * 2 + (size_t)2 * LAS_HEADS * (LAS_KEYS + 8) * 2;
}

struct LatentSplitParams {
  const __nv_bfloat16 *q_hi, *q_lo;  // [batch][heads][qrow]
  int qrow;
  const __nv_bfloat16* cache;        // [slot][cap][crow]
  int crow, kvp, cap;
  const int* positions;
  const int* slots;
  int heads, window, max_ctx, nsplit;
  float* part_o;                     // [batch][heads][nsplit][kvp]
  float* part_ml;                    // [batch][heads][nsplit]{max, sum}, base-e scores
};

// grid = (splits, groups of 16 heads, batch). TW = most 8-column tiles of the weighted sum per warp.
template <int TW>
__global__ void __launch_bounds__(LAS_THREADS) latent_split_kernel(const LatentSplitParams p) {
  extern __shared__ __align__(16) unsigned char las_smem[];
  __shared__ float mx_s[LAS_WARPS][LAS_HEADS], sum_s[LAS_WARPS][LAS_HEADS];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int split = blockIdx.x, h0 = blockIdx.y * LAS_HEADS, b = blockIdx.z;
  const int EP = las_row(p.crow), RS = EP + 8, PS = LAS_KEYS + 8;
  __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(las_smem);
  __nv_bfloat16* Qh = Ks + LAS_KEYS * RS;
  __nv_bfloat16* Ql = Qh + LAS_HEADS * RS;
  __nv_bfloat16* Ph = Ql + LAS_HEADS * RS;
  __nv_bfloat16* Pl = Ph + LAS_HEADS * PS;
  pdl_launch_dependents();
  pdl_wait();
  const int pos = p.positions[b];
  if (pos < 0 || pos >= p.max_ctx) return;
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0, nkeys = pos - lo + 1;
  const int chunk = ((nkeys + p.nsplit - 1) / p.nsplit + LAS_KEYS - 1) / LAS_KEYS * LAS_KEYS;
  const int k_begin = lo + split * chunk, k_end = min(pos + 1, k_begin + chunk);
  const __nv_bfloat16* cache = p.cache + (size_t)p.slots[b] * p.cap * p.crow;
  const int nh = min(LAS_HEADS, p.heads - h0), ce = EP >> 3, cc = p.crow >> 3;
  for (int r = warp; r < LAS_HEADS; r += LAS_WARPS) {
    const size_t at = ((size_t)b * p.heads + h0 + min(r, nh - 1)) * p.qrow;
    for (int c = lane; c < ce; c += 32) {
      if (r < nh) {
        pfa_cp16(Qh + r * RS + 8 * c, p.q_hi + at + 8 * c);
        pfa_cp16(Ql + r * RS + 8 * c, p.q_lo + at + 8 * c);
      } else {
        *reinterpret_cast<uint4*>(Qh + r * RS + 8 * c) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(Ql + r * RS + 8 * c) = make_uint4(0, 0, 0, 0);
      }
    }
  }
  const int tiles = p.kvp >> 3;  // 8-column tiles of the weighted sum; a warp takes pairs of them
  float o[TW][4];
#pragma unroll
  for (int i = 0; i < TW; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;  // heads g and g + 8
  for (int kt = k_begin; kt < k_end; kt += LAS_KEYS) {
    const int nk = min(LAS_KEYS, k_end - kt);
    __syncthreads();
    for (int r = warp; r < LAS_KEYS; r += LAS_WARPS) {
      const __nv_bfloat16* src = cache + (size_t)((kt + r) % p.cap) * p.crow;
      __nv_bfloat16* d = Ks + r * RS;
      for (int c = lane; c < ce; c += 32) {
        if (r < nk && c < cc) pfa_cp16(d + 8 * c, src + 8 * c);
        else *reinterpret_cast<uint4*>(d + 8 * c) = make_uint4(0, 0, 0, 0);
      }
    }
    pfa_cp_wait_all();
    __syncthreads();
    // scores of this warp's 8 keys
    float s[4] = {0.f, 0.f, 0.f, 0.f}, sl[4] = {0.f, 0.f, 0.f, 0.f};  // products with the queries' values and remainders
#pragma unroll 2
    for (int ks = 0; ks < EP; ks += 32) {
      uint32_t a0[4], a1[4], b0[4], b1[4], kb[4];
      const int aoff = (lane & 15) * RS + ks + (lane >> 4) * 8;
      pfa_ldm4(kb, Ks + (warp * 8 + (lane & 7)) * RS + ks + (lane >> 3) * 8);
      pfa_ldm4(a0, Qh + aoff);
      pfa_ldm4(a1, Qh + aoff + 16);
      pfa_ldm4(b0, Ql + aoff);
      pfa_ldm4(b1, Ql + aoff + 16);
      lap_mma(s, a0, kb[0], kb[1]);
      lap_mma(sl, b0, kb[0], kb[1]);
      lap_mma(s, a1, kb[2], kb[3]);
      lap_mma(sl, b1, kb[2], kb[3]);
    }
    float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool ok = warp * 8 + 2 * t + e < nk;
      s[e] = ok ? s[e] + sl[e] : -INFINITY;
      s[2 + e] = ok ? s[2 + e] + sl[2 + e] : -INFINITY;
      x0 = fmaxf(x0, s[e]);
      x1 = fmaxf(x1, s[2 + e]);
    }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
      x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, x));
      x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, x));
    }
    if (t == 0) { mx_s[warp][g] = x0; mx_s[warp][g + 8] = x1; }
    __syncthreads();
    float n0 = m0, n1 = m1;
#pragma unroll
    for (int w = 0; w < LAS_WARPS; ++w) {
      n0 = fmaxf(n0, mx_s[w][g]);
      n1 = fmaxf(n1, mx_s[w][g + 8]);
    }
    const float f0 = expf(m0 - n0), f1 = expf(m1 - n1);  // every tile has a key, so n is finite
    m0 = n0; m1 = n1;
    float y0 = 0.f, y1 = 0.f;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int k = warp * 8 + 2 * t + e;
      const float w0 = expf(s[e] - n0), w1 = expf(s[2 + e] - n1);
      y0 += w0; y1 += w1;
      split_bf16(w0, Ph[g * PS + k], Pl[g * PS + k]);
      split_bf16(w1, Ph[(g + 8) * PS + k], Pl[(g + 8) * PS + k]);
    }
    l0 = l0 * f0 + y0; l1 = l1 * f1 + y1;  // this thread's share; shares of lanes and warps are added at the end
#pragma unroll
    for (int i = 0; i < TW; ++i) { o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1; }
    __syncthreads();
    // weighted sums: this warp's pairs of column tiles
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      uint32_t ah[4], al[4];
      const int aoff = (lane & 15) * PS + kk * 16 + (lane >> 4) * 8;
      pfa_ldm4(ah, Ph + aoff);
      pfa_ldm4(al, Pl + aoff);
#pragma unroll
      for (int i = 0; i < TW / 2; ++i) {
        const int tile = 2 * (warp + LAS_WARPS * i);
        if (tile < tiles) {  // an odd last tile reads the row's next eight columns and drops them
          uint32_t vb[4];
          pfa_ldm4t(vb, Ks + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * RS + tile * 8 + (lane >> 4) * 8);
          lap_mma(o[2 * i], ah, vb[0], vb[1]);
          lap_mma(o[2 * i + 1], ah, vb[2], vb[3]);
          lap_mma(o[2 * i], al, vb[0], vb[1]);
          lap_mma(o[2 * i + 1], al, vb[2], vb[3]);
        }
      }
    }
  }
#pragma unroll
  for (int x = 1; x < 4; x <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, x);
    l1 += __shfl_xor_sync(0xffffffffu, l1, x);
  }
  __syncthreads();
  if (t == 0) { sum_s[warp][g] = l0; sum_s[warp][g + 8] = l1; mx_s[warp][g] = m0; mx_s[warp][g + 8] = m1; }
  __syncthreads();
  const size_t row = ((size_t)b * p.heads + h0) * p.nsplit + split;
  if (tid < nh) {
    float* ml = p.part_ml + (row + (size_t)tid * p.nsplit) * 2;
    ml[0] = mx_s[0][tid];
    float l = 0.f;
    for (int w = 0; w < LAS_WARPS; ++w) l += sum_s[w][tid];
    ml[1] = k_begin < k_end ? l : 0.f;
  }
  if (k_begin >= k_end) return;  // an empty run: its sum of zero makes the merge skip it
#pragma unroll
  for (int i = 0; i < TW; ++i) {
    const int tile = 2 * (warp + LAS_WARPS * (i >> 1)) + (i & 1);
    if (tile < tiles) {
      const int c = 8 * tile + 2 * t;
      if (g < nh) *reinterpret_cast<float2*>(p.part_o + (row + (size_t)g * p.nsplit) * p.kvp + c) = make_float2(o[i][0], o[i][1]);
      if (g + 8 < nh) *reinterpret_cast<float2*>(p.part_o + (row + (size_t)(g + 8) * p.nsplit) * p.kvp + c) = make_float2(o[i][2], o[i][3]);
    }
  }
}

constexpr int LAM_THREADS = 256, LAM_ROWS = 32;  // value rows per block: four per warp
constexpr int LAM_KEEP = 4;                      // pieces of each W_uv row a lane requests ahead (kv_rank up to 1024)

// grid = (vdim / 32 rounded up, heads, batch). O = type of the output rows.
template <typename O>
__global__ void __launch_bounds__(LAM_THREADS) latent_merge_kernel(const LatentDecodeParams p) {
  extern __shared__ __align__(16) float lam_s[];  // merged sum of latents [kvp], normalised
  __shared__ float w_s[LAD_MAX_SPLITS];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, b = blockIdx.z;
  const int r0 = blockIdx.x * LAM_ROWS + warp * 4, vch = p.kvp >> 3;
  pdl_launch_dependents();
  const __nv_bfloat16* uv = p.uv + (size_t)h * p.vdim * p.kvp;
  uint4 w[4][LAM_KEEP];
#pragma unroll
  for (int e = 0; e < 4; ++e)
#pragma unroll
    for (int i = 0; i < LAM_KEEP; ++i)
      w[e][i] = lane + 32 * i < vch && r0 + e < p.vdim ? ldg128(uv + (size_t)(r0 + e) * p.kvp + 8 * (lane + 32 * i)) : make_uint4(0, 0, 0, 0);
  pdl_wait();
  const int pos = p.positions[b];
  if (pos < 0 || pos >= p.max_ctx) return;
  const size_t base = ((size_t)b * p.heads + h) * p.nsplit;
  if (warp == 0) {  // weight of every run: exp(its max - the largest max) / total sum
    float m[LAD_MAX_SPLITS / 32], l[LAD_MAX_SPLITS / 32], M = -INFINITY, L = 0.f;
#pragma unroll
    for (int i = 0; i < LAD_MAX_SPLITS / 32; ++i) {
      const int s = lane + 32 * i;
      const float2 ml = s < p.nsplit ? __ldcg(reinterpret_cast<const float2*>(p.part_ml + (base + s) * 2)) : make_float2(0.f, 0.f);
      m[i] = ml.x; l[i] = ml.y;
      if (l[i] > 0.f) M = fmaxf(M, m[i]);
    }
    M = warp_max(M);
#pragma unroll
    for (int i = 0; i < LAD_MAX_SPLITS / 32; ++i) {
      m[i] = l[i] > 0.f ? expf(m[i] - M) : 0.f;
      L += m[i] * l[i];
    }
    L = warp_sum(L);
#pragma unroll
    for (int i = 0; i < LAD_MAX_SPLITS / 32; ++i) w_s[lane + 32 * i] = m[i] / L;
  }
  __syncthreads();
  for (int i = tid; i < p.kvp; i += LAM_THREADS) {
    float o = 0.f;
#pragma unroll 16
    for (int s = 0; s < p.nsplit; ++s) {
      const float v = __ldcg(p.part_o + (base + s) * p.kvp + i);
      o = w_s[s] > 0.f ? fmaf(w_s[s], v, o) : o;  // an empty run's row was never written
    }
    lam_s[i] = o;
  }
  __syncthreads();
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  auto add = [&](int e, const uint4& u, const float* x) {
    acc[e] = fmaf(bf_lo(u.x), x[0], acc[e]); acc[e] = fmaf(bf_hi(u.x), x[1], acc[e]); acc[e] = fmaf(bf_lo(u.y), x[2], acc[e]); acc[e] = fmaf(bf_hi(u.y), x[3], acc[e]);
    acc[e] = fmaf(bf_lo(u.z), x[4], acc[e]); acc[e] = fmaf(bf_hi(u.z), x[5], acc[e]); acc[e] = fmaf(bf_lo(u.w), x[6], acc[e]); acc[e] = fmaf(bf_hi(u.w), x[7], acc[e]);
  };
#pragma unroll
  for (int i = 0; i < LAM_KEEP; ++i)
    if (lane + 32 * i < vch) {
      float x[8];
      load8(lam_s + 8 * (lane + 32 * i), x);
#pragma unroll
      for (int e = 0; e < 4; ++e) add(e, w[e][i], x);
    }
  for (int c = lane + 32 * LAM_KEEP; c < vch; c += 32) {
    float x[8];
    load8(lam_s + 8 * c, x);
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (r0 + e < p.vdim) add(e, ldg128(uv + (size_t)(r0 + e) * p.kvp + 8 * c), x);
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) acc[e] = warp_sum(acc[e]);
  if (lane < 4 && r0 + lane < p.vdim) {
    const float v = lane == 0 ? acc[0] : lane == 1 ? acc[1] : lane == 2 ? acc[2] : acc[3];
    const int j = h * p.vdim + r0 + lane;
    static_cast<O*>(p.out)[(size_t)b * p.out_stride + j] = to_operand<O>(v * p.gate[(size_t)b * p.gate_stride + j]);
  }
}

// ---- prompts -----------------------------------------------------------------------------------------------------
constexpr int LAP_Q = 128, LAP_K = 64, LAP_THREADS = 256, LAP_WARPS = 8;

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
__host__ __device__ __forceinline__ int lap_value_cols(int vdim) { return vdim <= 32 ? 32 : vdim <= 64 ? 64 : vdim <= 128 ? 128 : 256; }
__host__ __device__ __forceinline__ size_t lap_smem_bytes(int dim, int rot, int vp) {
  return ((size_t)(LAP_Q + LAP_K) * lap_qk_stride(dim, rot) + (size_t)LAP_K * (vp + 8)) * 2;
}

// grid = (query blocks of the longest run, heads, runs). VP = value columns per head rounded up to 32, 64, 128 or 256.
template <int VP>
__global__ void __launch_bounds__(LAP_THREADS, VP <= 128 ? 2 : 1) latent_prefill_kernel(const LatentPrefillParams p) {
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
  const bool vec = !((p.dim | p.rot_dim | p.vdim | p.kv_stride | p.v_off | p.kr_stride | p.q_stride) & 7);
  // queries, rotated; the scale is applied to the products
  if (vec) {  // pieces of four elements (two pairs), eight of them in flight per thread
    const int n4 = EP >> 2, d4 = p.dim >> 2, e4 = E >> 2;
    for (int i0 = tid; i0 < LAP_Q * n4; i0 += 8 * LAP_THREADS) {
      float4 v[8], cs[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int i = i0 + k * LAP_THREADS, r = i / n4, c = i - r * n4;
        const bool ok = r < nq && c < e4;
        v[k] = ok ? *reinterpret_cast<const float4*>(p.q + (size_t)(run.row0 + q0 + r) * p.q_stride + h * E + 4 * c) : make_float4(0.f, 0.f, 0.f, 0.f);
        cs[k] = make_float4(1.f, 0.f, 1.f, 0.f);  // pairs beyond the rotated ones pass
        const int j = 2 * (c - d4);               // first of the piece's two pairs
        if (ok && j >= 0) {
          const float* table = p.rope + ((size_t)(run.start + q0 + r) * p.pairs + j) * 2;
          if (j < p.pairs) { cs[k].x = table[0]; cs[k].y = table[1]; }
          if (j + 1 < p.pairs) { cs[k].z = table[2]; cs[k].w = table[3]; }
        }
      }
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int i = i0 + k * LAP_THREADS, r = i / n4, c = i - r * n4;
        if (r < LAP_Q)
          *reinterpret_cast<uint2*>(Qs + r * QS + 4 * c) = make_uint2(pack_bf2(v[k].x * cs[k].x - v[k].y * cs[k].y, v[k].y * cs[k].x + v[k].x * cs[k].y),
                                                                      pack_bf2(v[k].z * cs[k].z - v[k].w * cs[k].w, v[k].w * cs[k].z + v[k].z * cs[k].w));
      }
    }
  } else {
    for (int r = warp; r < LAP_Q; r += LAP_WARPS) {
      const float* qr = p.q + (size_t)(run.row0 + q0 + min(r, nq - 1)) * p.q_stride + h * E;
      const float* table = p.rope + (size_t)(run.start + q0 + min(r, nq - 1)) * p.pairs * 2;
      for (int c = lane; c < EP; c += 32) {
        float v = 0.f;
        if (r < nq && c < E) v = c < p.dim ? qr[c] : rotated(qr + p.dim, c - p.dim, table, p.pairs);
        Qs[r * QS + c] = __float2bfloat16(v);
      }
    }
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

  // Key and value tiles have one buffer each: the next key tile is requested as soon as this one's scores are done, the
  // next value tile after this one's products, so each copy runs under the other half of the work.
  auto load_k = [&](int kt) {
    const int nk = min(LAP_K, klast - kt + 1);
    const size_t crow = (size_t)(run.ctx0 + kt - base);
    if (vec) {
      const int ce = EP >> 3, cd = p.dim >> 3, cn = E >> 3;
      for (int r = warp; r < LAP_K; r += LAP_WARPS) {
        const __nv_bfloat16* kv = p.kv + (crow + r) * p.kv_stride + h * p.dim;
        const __nv_bfloat16* kr = p.kr + (crow + r) * p.kr_stride;
        for (int c = lane; c < ce; c += 32) {
          __nv_bfloat16* d = Ks + r * QS + 8 * c;
          if (r < nk && c < cn) pfa_cp16(d, c < cd ? kv + 8 * c : kr + 8 * (c - cd));
          else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
        }
      }
    } else {
      for (int i = tid; i < LAP_K * EP; i += LAP_THREADS) {
        const int r = i / EP, c = i - r * EP;
        __nv_bfloat16 v = __float2bfloat16(0.f);
        if (r < nk && c < E) v = c < p.dim ? p.kv[(crow + r) * p.kv_stride + h * p.dim + c] : p.kr[(crow + r) * p.kr_stride + c - p.dim];
        Ks[r * QS + c] = v;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto load_v = [&](int kt) {
    const int nk = min(LAP_K, klast - kt + 1);
    const size_t crow = (size_t)(run.ctx0 + kt - base);
    if (vec) {
      constexpr int CV = VP >> 3;
      const int cvn = p.vdim >> 3;
      for (int i = tid; i < LAP_K * CV; i += LAP_THREADS) {
        const int r = i / CV, c = i % CV;
        __nv_bfloat16* d = Vs + r * VS + 8 * c;
        if (r < nk && c < cvn) pfa_cp16(d, p.kv + (crow + r) * p.kv_stride + p.v_off + h * p.vdim + 8 * c);
        else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
      }
    } else {
      for (int i = tid; i < LAP_K * VP; i += LAP_THREADS) {
        const int r = i / VP, c = i - r * VP;
        Vs[r * VS + c] = r < nk && c < p.vdim ? p.kv[(crow + r) * p.kv_stride + p.v_off + h * p.vdim + c] : __float2bfloat16(0.f);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load_k(kfirst);
  load_v(kfirst);
  for (int kt = kfirst; kt <= klast; kt += LAP_K) {
    asm volatile("cp.async.wait_group 1;" ::: "memory");  // the key tile; its value tile may still be on its way
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
    __syncthreads();  // every warp has read the key tile
    if (kt + LAP_K <= klast) load_k(kt + LAP_K);
    else asm volatile("cp.async.commit_group;" ::: "memory");  // keeps one group per step
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
    asm volatile("cp.async.wait_group 1;" ::: "memory");  // the value tile
    __syncthreads();
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
    __syncthreads();  // every warp has read the value tile
    if (kt + LAP_K <= klast) load_v(kt + LAP_K);
    else asm volatile("cp.async.commit_group;" ::: "memory");
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
