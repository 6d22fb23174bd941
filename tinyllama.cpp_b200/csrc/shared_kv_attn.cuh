// Shared-kv attention: grouped-query attention whose values are its keys as they were projected; only queries and keys are
// rotated, over their first 2 * pairs dimensions. Scores may be capped (cap * tanh(s / cap)), the softmax may have a sink (one
// more term exp(0) in the denominator, without a value), and any KeyMask applies. The cache keeps one row per token and
// key / value head: [key as projected, padded to 8 | its rotated dimensions, padded to 8], so values are the row's first part
// and a score is the product of (rest of the query, rotated query) with (rest of the first part, second part). Per slot and
// head the rows are a ring of `cap` (position p in row p % cap), cap >= mask size - 1 + tokens per launch.
//
//   shared_kv_append_kernel  prompts: rows of the new tokens into the rings, which prompt_attn_kernel then reads directly
//   shared_kv_decode_kernel  one token of several sequences, bfloat16 cache: rotation, append, scores and weighted sums of up
//                            to 16 query heads of one key / value head over a run of keys (split_attend), and the merge of
//                            the runs by the block that finishes last, in one launch
//   shared_kv_rows_kernel    32-bit engines, one query head of one token per block, over rows that are in the cache already
//
// A = type of the cache and of matmul operands: __nv_bfloat16, or float in a 32-bit engine.
#pragma once
#include "attn_tiles.cuh"

namespace b200 {

constexpr int SKV_MAX_SPLITS = 64;

struct SharedKvParams {
  const float* q;       // [rows][q_stride]: heads * dim, unrotated
  int q_stride;
  const float* k;       // [rows][k_stride]: kv_heads * dim, the new tokens' keys as projected
  int k_stride;
  const float* rope;    // [max_ctx][pairs]{cos, sin}
  int pairs;
  void* cache;          // [slot][kv_heads][cap][crow]
  int vp, crow, cap;    // vp = pad8(dim), crow = vp + pad8(2 * pairs)
  const int* positions;
  const int* slots;
  int rows, heads, kv_heads, dim, max_ctx;
  KeyMask mask;
  float scale, softcap;
  int sink;
  int nsplit;           // context splits per (head group, sequence)
  float* part_o;        // [batch][heads][nsplit][vp]
  float* part_ml;       // [batch][heads][nsplit]{max, sum}
  int* tickets;         // [batch][head groups], zero between launches
  void* out;            // [rows][out_stride]: FP32 rows, or matmul operands when out_bf16 is set
  int out_stride, out_bf16;
  int* error_flag;
};

// Head groups of a decode launch: up to 16 query heads that share a key / value head.
__host__ __device__ __forceinline__ int skv_groups(int heads, int kv_heads) { return kv_heads * ((heads / kv_heads + LAS_HEADS - 1) / LAS_HEADS); }

// Column i of a cache row made from a projected key: the key itself, then its rotated dimensions.
__device__ __forceinline__ float skv_row(const SharedKvParams& p, const float* key, const float* table, int i) {
  if (i < p.vp) return i < p.dim ? key[i] : 0.f;
  return i - p.vp < 2 * p.pairs ? rotated(key, i - p.vp, table, p.pairs) : 0.f;
}
// The query in the layout of a cache row: nothing where the key's unrotated copy of a rotated dimension lies.
__device__ __forceinline__ float skv_query(const SharedKvParams& p, const float* q, const float* table, int i) {
  if (i < p.vp) return i >= 2 * p.pairs && i < p.dim ? q[i] : 0.f;
  return i - p.vp < 2 * p.pairs ? rotated(q, i - p.vp, table, p.pairs) : 0.f;
}

// One warp per (row, key / value head).
template <typename A>
__global__ void __launch_bounds__(256) shared_kv_append_kernel(const SharedKvParams p) {
  const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= p.rows * p.kv_heads) return;
  const int t = item / p.kv_heads, g = item - t * p.kv_heads, pos = p.positions[t];
  if (pos < 0 || pos >= p.max_ctx) {  // nothing is appended
    if (lane == 0 && p.error_flag) *reinterpret_cast<volatile int*>(p.error_flag) = 3;
    return;
  }
  const float* key = p.k + (size_t)t * p.k_stride + g * p.dim;
  const float* table = p.rope + (size_t)pos * p.pairs * 2;
  A* row = static_cast<A*>(p.cache) + (((size_t)p.slots[t] * p.kv_heads + g) * p.cap + pos % p.cap) * p.crow;
  for (int i = lane; i < p.crow; i += 32) row[i] = to_operand<A>(skv_row(p, key, table, i));
}

// grid = (splits, head groups, batch). TW = most 8-column tiles of the weighted sum per warp, O = type of the output rows.
template <int TW, typename O>
__global__ void __launch_bounds__(LAS_THREADS) shared_kv_decode_kernel(const SharedKvParams p) {
  extern __shared__ __align__(16) unsigned char skv_smem[];
  __shared__ SplitStats st;
  __shared__ float w_s[LAS_HEADS][SKV_MAX_SPLITS];  // weight of every run of a head
  __shared__ int last_s;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int split = blockIdx.x, b = blockIdx.z, per = p.heads / p.kv_heads, sub = gridDim.y / p.kv_heads;
  const int g = blockIdx.y / sub, part = blockIdx.y - g * sub;  // key / value head, and which 16 of its query heads
  const int h0 = g * per + part * LAS_HEADS, nh = min(LAS_HEADS, per - part * LAS_HEADS);
  const SplitTiles m(skv_smem, p.crow);
  pdl_launch_dependents();
  pdl_wait();
  const int pos = p.positions[b], slot = p.slots[b];
  if (pos < 0 || pos >= p.max_ctx) {  // nothing is read or appended for this sequence
    if (tid == 0 && p.error_flag) *reinterpret_cast<volatile int*>(p.error_flag) = 3;
    return;
  }
  const int lo = p.mask.first(pos), nkeys = pos - lo + 1;
  const int chunk = ((nkeys + p.nsplit - 1) / p.nsplit + LAS_KEYS - 1) / LAS_KEYS * LAS_KEYS;
  const int k_begin = lo + split * chunk, k_end = min(pos + 1, k_begin + chunk);
  const int ce = m.EP >> 3, cc = p.crow >> 3;
  __nv_bfloat16* cache = static_cast<__nv_bfloat16*>(p.cache) + ((size_t)slot * p.kv_heads + g) * p.cap * p.crow;
  const float* table = p.rope + (size_t)pos * p.pairs * 2;
  auto queries = [&] {
    const int pieces = m.EP / 32;  // of 32 columns; those of the group's heads are shared out evenly over the warps
    const float* q = p.q + (size_t)b * p.q_stride + (size_t)h0 * p.dim;
#pragma unroll 4
    for (int i = warp; i < nh * pieces; i += LAS_WARPS) {
      const int r = i / pieces, c = (i - r * pieces) * 32 + lane;
      split_bf16(c < p.crow ? skv_query(p, q + r * p.dim, table, c) * p.scale : 0.f, m.Qh[r * m.RS + c], m.Ql[r * m.RS + c]);
    }
    for (int i = nh * ce + tid; i < LAS_HEADS * ce; i += LAS_THREADS) {
      const int r = i / ce, c = i - r * ce;
      *reinterpret_cast<uint4*>(m.Qh + r * m.RS + 8 * c) = *reinterpret_cast<uint4*>(m.Ql + r * m.RS + 8 * c) = make_uint4(0, 0, 0, 0);
    }
  };
  // the new token's row is made here, by every block whose run it lies in; one of them keeps it
  const int ring0 = k_begin % p.cap;
  const float* key = p.k + (size_t)b * p.k_stride + g * p.dim;
  auto load_row = [&](int kp, __nv_bfloat16* d) {
    const int at = ring0 + kp - k_begin;  // fewer rows than the ring has: it wraps once at most
    __nv_bfloat16* row = cache + (size_t)(at >= p.cap ? at - p.cap : at) * p.crow;
    if (kp == pos) {
      for (int c = lane; c < m.EP; c += 32) {
        const __nv_bfloat16 v = __float2bfloat16(c < p.crow ? skv_row(p, key, table, c) : 0.f);
        d[c] = v;
        if (part == 0 && c < p.crow) row[c] = v;
      }
      return;
    }
    for (int c = lane; c < ce; c += 32) {
      if (c < cc) pfa_cp16(d + 8 * c, row + 8 * c);
      else *reinterpret_cast<uint4*>(d + 8 * c) = make_uint4(0, 0, 0, 0);
    }
  };
  const int tiles = p.vp >> 3;
  float o[TW][4];
  const float to_tanh = p.softcap > 0.f ? 2.8853900817779268f / p.softcap : 0.f;
  auto score = [&](float s) { return p.softcap > 0.f ? fmaf(-2.f * p.softcap, rcp_fast(1.f + ex2_fast(s * to_tanh)), p.softcap) : s; };  // as in prompt_attn_kernel
  // whole 32-column steps in which every query is zero are left out
  split_attend<TW>(m, st, k_begin, k_end, 2 * p.pairs / 32 * 32, tiles, queries, load_row, score, o);

  auto put = [&](int h, int c, float v) {
    if (c < p.dim) static_cast<O*>(p.out)[(size_t)b * p.out_stride + (size_t)(h0 + h) * p.dim + c] = to_operand<O>(v);
  };
  float total = 0.f;
  if (tid < nh && k_begin < k_end)
    for (int w = 0; w < LAS_WARPS; ++w) total += st.sum[w][tid];
  if (p.nsplit == 1) {
    if (tid < nh) {
      const float mx = st.mx[0][tid], M = p.sink ? fmaxf(mx, 0.f) : mx, f = expf(mx - M);
      w_s[tid][0] = f / (f * total + (p.sink ? expf(-M) : 0.f));
    }
    __syncthreads();
    split_columns<TW>(o, tiles, nh, [&](int h, int c, float x, float y) { put(h, c, x * w_s[h][0]); put(h, c + 1, y * w_s[h][0]); });
    return;
  }
  const size_t base = ((size_t)b * p.heads + h0) * p.nsplit;  // head h0 + h, run s: base + h * nsplit + s
  if (tid < nh) *reinterpret_cast<float2*>(p.part_ml + (base + (size_t)tid * p.nsplit + split) * 2) = make_float2(st.mx[0][tid], total);
  if (k_begin < k_end)
    split_columns<TW>(o, tiles, nh, [&](int h, int c, float x, float y) {
      *reinterpret_cast<float2*>(p.part_o + (base + (size_t)h * p.nsplit + split) * p.vp + c) = make_float2(x, y);
    });
  __syncthreads();
  int* ticket = p.tickets + (size_t)b * gridDim.y + blockIdx.y;
  if (tid == 0) {  // the fence covers what the block's other threads wrote before the barrier
    __threadfence();
    last_s = atomicAdd(ticket, 1) == p.nsplit - 1;
    __threadfence();
  }
  __syncthreads();
  if (!last_s) return;
  if (tid == 0) *ticket = 0;
  for (int h = warp; h < nh; h += LAS_WARPS) {  // weight of every run: exp(its max - the largest max) / total sum
    float mx[SKV_MAX_SPLITS / 32], l[SKV_MAX_SPLITS / 32], M = p.sink ? 0.f : -INFINITY, L = 0.f;
#pragma unroll
    for (int i = 0; i < SKV_MAX_SPLITS / 32; ++i) {
      const int s = lane + 32 * i;
      const float2 ml = s < p.nsplit ? __ldcg(reinterpret_cast<const float2*>(p.part_ml + (base + (size_t)h * p.nsplit + s) * 2)) : make_float2(0.f, 0.f);
      mx[i] = ml.x; l[i] = ml.y;
      if (l[i] > 0.f) M = fmaxf(M, mx[i]);
    }
    M = warp_max(M);
#pragma unroll
    for (int i = 0; i < SKV_MAX_SPLITS / 32; ++i) {
      mx[i] = l[i] > 0.f ? expf(mx[i] - M) : 0.f;
      L += mx[i] * l[i];
    }
    L = warp_sum(L) + (p.sink ? expf(-M) : 0.f);
#pragma unroll
    for (int i = 0; i < SKV_MAX_SPLITS / 32; ++i) w_s[h][lane + 32 * i] = mx[i] / L;
  }
  __syncthreads();
  const int used = (nkeys + chunk - 1) / chunk;  // the runs that have keys
  for (int i = tid; i < nh * p.vp; i += LAS_THREADS) {
    const int h = i / p.vp, c = i - h * p.vp;
    const float* src = p.part_o + (base + (size_t)h * p.nsplit) * p.vp + c;
    float v = 0.f;
#pragma unroll 8
    for (int s = 0; s < used; ++s) v = fmaf(w_s[h][s], __ldcg(src + (size_t)s * p.vp), v);
    put(h, c, v);
  }
}

constexpr int SKR_THREADS = 128, SKR_KEYS = 128;
__host__ __device__ __forceinline__ size_t skr_smem_bytes(int crow, int vp) { return (size_t)(crow + vp) * 4; }

// FP32 throughout: keys in tiles of 128 with an online softmax. grid = (heads, rows).
__global__ void __launch_bounds__(SKR_THREADS) shared_kv_rows_kernel(const SharedKvParams p) {
  extern __shared__ __align__(16) float skr_s[];  // query (crow) | weighted sum (vp)
  __shared__ float sc[SKR_KEYS], red[SKR_THREADS / 32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, t = blockIdx.y, g = h / (p.heads / p.kv_heads);
  float *qv = skr_s, *ol = qv + p.crow;
  const int pos = p.positions[t];
  if (pos < 0 || pos >= p.max_ctx) return;
  const float* cache = static_cast<const float*>(p.cache) + ((size_t)p.slots[t] * p.kv_heads + g) * p.cap * p.crow;
  const float* q = p.q + (size_t)t * p.q_stride + (size_t)h * p.dim;
  const float* table = p.rope + (size_t)pos * p.pairs * 2;
  for (int i = tid; i < p.crow; i += SKR_THREADS) qv[i] = skv_query(p, q, table, i);
  for (int i = tid; i < p.vp; i += SKR_THREADS) ol[i] = 0.f;
  float M = p.sink ? 0.f : -INFINITY, L = p.sink ? 1.f : 0.f;
  __syncthreads();
  for (int k0 = p.mask.first(pos); k0 <= pos; k0 += SKR_KEYS) {
    const int n = min(SKR_KEYS, pos + 1 - k0);
    float mx = -INFINITY;
    for (int k = warp; k < n; k += SKR_THREADS / 32) {
      const float* row = cache + (size_t)((k0 + k) % p.cap) * p.crow;
      float s = 0.f;
      for (int i = lane; i < p.crow; i += 32) s = fmaf(qv[i], row[i], s);
      s = capped_score(warp_sum(s) * p.scale, p.softcap);
      if (lane == 0) sc[k] = s;
      mx = fmaxf(mx, s);
    }
    if (lane == 0) red[warp] = mx;
    __syncthreads();
    float N = M;
#pragma unroll
    for (int w = 0; w < SKR_THREADS / 32; ++w) N = fmaxf(N, red[w]);
    const float f = expf(M - N);
    M = N;
    __syncthreads();
    float sum[1] = {0.f};
    for (int k = tid; k < n; k += SKR_THREADS) {
      const float e = expf(sc[k] - N);
      sc[k] = e;
      sum[0] += e;
    }
    block_sums<1, SKR_THREADS / 32>(sum, red);
    L = L * f + sum[0];
    for (int c = tid; c < p.vp; c += SKR_THREADS) {
      float v = ol[c] * f;
      for (int k = 0; k < n; ++k) v = fmaf(sc[k], cache[(size_t)((k0 + k) % p.cap) * p.crow + c], v);
      ol[c] = v;
    }
    __syncthreads();
  }
  for (int c = tid; c < p.dim; c += SKR_THREADS) static_cast<float*>(p.out)[(size_t)t * p.out_stride + (size_t)h * p.dim + c] = ol[c] / L;
}

}  // namespace b200
