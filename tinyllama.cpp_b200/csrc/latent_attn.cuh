// Latent attention: keys and values of all heads are linear images of one small vector c per token (kv_rank elements,
// RMS-normed), plus one rotated key part of rot_dim elements shared by the heads. The cache holds only [c | rotated
// part] per token, in rows padded to multiples of 8 elements; a sliding window keeps the cache a ring of `cap` rows
// (position p in row p % cap), cap >= window - 1 + tokens per launch.
//
//   latent_append_kernel   prompts: norm + rotation of new rows into the ring, and the rows a chunk attends to laid out
//                          contiguously (history from the ring, then the new ones) for the key / value expansion
//                          that prompt_attn_kernel (attn_tiles.cuh) then runs over
//   decode                 one token of several sequences: works on the latents themselves. The query's unrotated part is
//                          taken through W_uk once (q . W_uk c = (W_uk^T q) . c), scores and the weighted sum run over c,
//                          and the sum is taken through W_uv at the end. latent_decode_kernel does all of it for one
//                          head in FP32 (32-bit engines); bfloat16 engines split it into three launches
//                          (latent_absorb_kernel, latent_split_kernel, latent_merge_kernel)
//
// A = type of the cache and of matmul operands: __nv_bfloat16, or float in a 32-bit engine.
#pragma once
#include "attn_tiles.cuh"

namespace b200 {

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
  int heads, dim, rot_dim, vdim, kv_rank, max_ctx;
  KeyMask mask;
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
  const int lo = p.mask.first(pos), nkeys = pos - lo + 1;
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

// ---- decode on the tensor cores (bfloat16 cache) -------------------------------------------------------------------
// Three launches: latent_absorb_kernel takes the queries through W_uk and appends the new rows, latent_split_kernel runs
// scores and weighted sums for 16 heads and one run of keys per block (split_attend), latent_merge_kernel merges the runs
// and goes through W_uv.

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

struct LatentSplitParams {
  const __nv_bfloat16 *q_hi, *q_lo;  // [batch][heads][qrow]
  int qrow;
  const __nv_bfloat16* cache;        // [slot][cap][crow]
  int crow, kvp, cap;
  const int* positions;
  const int* slots;
  int heads, max_ctx, nsplit;
  KeyMask mask;
  float* part_o;                     // [batch][heads][nsplit][kvp]
  float* part_ml;                    // [batch][heads][nsplit]{max, sum}, base-e scores
};

// grid = (splits, groups of 16 heads, batch). TW = most 8-column tiles of the weighted sum per warp.
template <int TW>
__global__ void __launch_bounds__(LAS_THREADS) latent_split_kernel(const LatentSplitParams p) {
  extern __shared__ __align__(16) unsigned char las_smem[];
  __shared__ SplitStats st;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int split = blockIdx.x, h0 = blockIdx.y * LAS_HEADS, b = blockIdx.z;
  const SplitTiles m(las_smem, p.crow);
  pdl_launch_dependents();
  pdl_wait();
  const int pos = p.positions[b];
  if (pos < 0 || pos >= p.max_ctx) return;
  const int lo = p.mask.first(pos), nkeys = pos - lo + 1;
  const int chunk = ((nkeys + p.nsplit - 1) / p.nsplit + LAS_KEYS - 1) / LAS_KEYS * LAS_KEYS;
  const int k_begin = lo + split * chunk, k_end = min(pos + 1, k_begin + chunk);
  const __nv_bfloat16* cache = p.cache + (size_t)p.slots[b] * p.cap * p.crow;
  const int nh = min(LAS_HEADS, p.heads - h0), ce = m.EP >> 3, cc = p.crow >> 3;
  auto queries = [&] {
    for (int r = warp; r < LAS_HEADS; r += LAS_WARPS) {
      const size_t at = ((size_t)b * p.heads + h0 + min(r, nh - 1)) * p.qrow;
      for (int c = lane; c < ce; c += 32) {
        if (r < nh) {
          pfa_cp16(m.Qh + r * m.RS + 8 * c, p.q_hi + at + 8 * c);
          pfa_cp16(m.Ql + r * m.RS + 8 * c, p.q_lo + at + 8 * c);
        } else {
          *reinterpret_cast<uint4*>(m.Qh + r * m.RS + 8 * c) = make_uint4(0, 0, 0, 0);
          *reinterpret_cast<uint4*>(m.Ql + r * m.RS + 8 * c) = make_uint4(0, 0, 0, 0);
        }
      }
    }
  };
  const int tiles = p.kvp >> 3;  // 8-column tiles of the weighted sum; a warp takes pairs of them
  float o[TW][4];
  auto load_row = [&](int key, __nv_bfloat16* d) {
    const __nv_bfloat16* src = cache + (size_t)(key % p.cap) * p.crow;
    for (int c = lane; c < ce; c += 32) {
      if (c < cc) pfa_cp16(d + 8 * c, src + 8 * c);
      else *reinterpret_cast<uint4*>(d + 8 * c) = make_uint4(0, 0, 0, 0);
    }
  };
  split_attend<TW>(m, st, k_begin, k_end, 0, tiles, queries, load_row, [](float s) { return s; }, o);
  const size_t row = ((size_t)b * p.heads + h0) * p.nsplit + split;
  if (tid < nh) {
    float* ml = p.part_ml + (row + (size_t)tid * p.nsplit) * 2;
    ml[0] = st.mx[0][tid];
    float l = 0.f;
    for (int w = 0; w < LAS_WARPS; ++w) l += st.sum[w][tid];
    ml[1] = k_begin < k_end ? l : 0.f;
  }
  if (k_begin >= k_end) return;  // an empty run: its sum of zero makes the merge skip it
  split_columns<TW>(o, tiles, nh, [&](int h, int c, float x, float y) {
    *reinterpret_cast<float2*>(p.part_o + (row + (size_t)h * p.nsplit) * p.kvp + c) = make_float2(x, y);
  });
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

}  // namespace b200
