// Pieces of the block models' attention kernels that do not depend on where keys and values come from: masks, score caps,
// the tensor-core decode of up to 16 heads over a run of keys (split_attend), and prompt attention (prompt_attn_kernel).
//
// A = type of the cache and of matmul operands: __nv_bfloat16, or float in a 32-bit engine.
#pragma once
#include "attn_prefill.cuh"
#include "block_rows.cuh"

namespace b200 {

// Which keys a query sees: all up to its own position (size 0), the last `size` positions, or (chunked) those of its own
// block of `size` positions counted from position 0.
struct KeyMask {
  int size, chunked;
  __host__ __device__ __forceinline__ int first(int pos) const {
    if (size <= 0) return 0;
    if (chunked) return pos - pos % size;
    return pos >= size ? pos - size + 1 : 0;
  }
};

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

// cap * tanh(s / cap), or s itself without a cap
__device__ __forceinline__ float capped_score(float s, float cap) { return cap > 0.f ? cap * tanhf(s / cap) : s; }

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

// ---- decode on the tensor cores -------------------------------------------------------------------------------------
// The cached rows are bfloat16 as they are; queries and attention weights enter the products as the sum of two bfloat16
// numbers (value and remainder), so that they keep 16 bits of mantissa and the scores FP32 character.

__device__ __forceinline__ void split_bf16(float v, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16(v);
  lo = __float2bfloat16(v - __bfloat162float(hi));
}

constexpr int LAS_THREADS = 256, LAS_WARPS = 8, LAS_HEADS = 16, LAS_KEYS = 64;

__host__ __device__ __forceinline__ int las_row(int n) { return (n + 31) / 32 * 32; }
__host__ __device__ __forceinline__ size_t las_smem_bytes(int crow) {
  const size_t row = las_row(crow) + 8;
  return (LAS_KEYS + 2 * LAS_HEADS) * row * 2 + (size_t)2 * LAS_HEADS * (LAS_KEYS + 8) * 2;
}


// Shared memory of a block: rows of 64 keys, the queries of 16 heads, the weights of a tile.
struct SplitTiles {
  __nv_bfloat16 *Ks, *Qh, *Ql, *Ph, *Pl;
  int EP, RS;  // columns of a row (a multiple of 32), row stride
  __device__ __forceinline__ SplitTiles(unsigned char* smem, int crow) : EP(las_row(crow)), RS(EP + 8) {
    Ks = reinterpret_cast<__nv_bfloat16*>(smem);
    Qh = Ks + LAS_KEYS * RS;
    Ql = Qh + LAS_HEADS * RS;
    Ph = Ql + LAS_HEADS * RS;
    Pl = Ph + LAS_HEADS * (LAS_KEYS + 8);
  }
};
// Running maximum of every head per warp, and the sums: after split_attend the final ones.
struct SplitStats {
  float mx[LAS_WARPS][LAS_HEADS], sum[LAS_WARPS][LAS_HEADS];
};

// Scores and weighted sums of 16 heads over the keys k_begin .. k_end - 1 (64 at a time), online softmax. load_row(key, dst)
// brings a key's row into shared memory, one warp per row (columns beyond the row must come out as zeros; cp.async allowed);
// scores run over columns ks0 .., the weighted sum over the first 8 * tiles columns: o[i] = this warp's column tile
// 2 (warp + 8 (i / 2)) + i % 2 for heads g and g + 8. score(s) turns a product into a score. Ends with a block barrier, the
// statistics complete in st (sums per warp; every warp holds the same maxima). queries() fills Qh and Ql; it runs while the
// first rows are on their way.
template <int TW, typename Queries, typename LoadRow, typename Score>
__device__ __forceinline__ void split_attend(const SplitTiles& m, SplitStats& st, int k_begin, int k_end, int ks0, int tiles, Queries queries, LoadRow load_row,
                                             Score score, float (&o)[TW][4]) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int RS = m.RS, PS = LAS_KEYS + 8;
#pragma unroll
  for (int i = 0; i < TW; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;  // heads g and g + 8
  for (int kt = k_begin; kt < k_end; kt += LAS_KEYS) {
    const int nk = min(LAS_KEYS, k_end - kt);
    if (kt > k_begin) __syncthreads();
    for (int r = warp; r < LAS_KEYS; r += LAS_WARPS) {
      __nv_bfloat16* d = m.Ks + r * RS;
      if (r < nk) load_row(kt + r, d);
      else
        for (int c = lane; c < m.EP >> 3; c += 32) *reinterpret_cast<uint4*>(d + 8 * c) = make_uint4(0, 0, 0, 0);
    }
    if (kt == k_begin) queries();
    pfa_cp_wait_all();
    __syncthreads();
    // scores of this warp's 8 keys
    float s[4] = {0.f, 0.f, 0.f, 0.f}, sl[4] = {0.f, 0.f, 0.f, 0.f};  // products with the queries' values and remainders
#pragma unroll 2
    for (int ks = ks0; ks < m.EP; ks += 32) {
      uint32_t a0[4], a1[4], b0[4], b1[4], kb[4];
      const int aoff = (lane & 15) * RS + ks + (lane >> 4) * 8;
      pfa_ldm4(kb, m.Ks + (warp * 8 + (lane & 7)) * RS + ks + (lane >> 3) * 8);
      pfa_ldm4(a0, m.Qh + aoff);
      pfa_ldm4(a1, m.Qh + aoff + 16);
      pfa_ldm4(b0, m.Ql + aoff);
      pfa_ldm4(b1, m.Ql + aoff + 16);
      lap_mma(s, a0, kb[0], kb[1]);
      lap_mma(sl, b0, kb[0], kb[1]);
      lap_mma(s, a1, kb[2], kb[3]);
      lap_mma(sl, b1, kb[2], kb[3]);
    }
    float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool ok = warp * 8 + 2 * t + e < nk;
      s[e] = ok ? score(s[e] + sl[e]) : -INFINITY;
      s[2 + e] = ok ? score(s[2 + e] + sl[2 + e]) : -INFINITY;
      x0 = fmaxf(x0, s[e]);
      x1 = fmaxf(x1, s[2 + e]);
    }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
      x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, x));
      x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, x));
    }
    if (t == 0) { st.mx[warp][g] = x0; st.mx[warp][g + 8] = x1; }
    __syncthreads();
    float n0 = m0, n1 = m1;
#pragma unroll
    for (int w = 0; w < LAS_WARPS; ++w) {
      n0 = fmaxf(n0, st.mx[w][g]);
      n1 = fmaxf(n1, st.mx[w][g + 8]);
    }
    const float f0 = expf(m0 - n0), f1 = expf(m1 - n1);  // every tile has a key, so n is finite
    m0 = n0; m1 = n1;
    float y0 = 0.f, y1 = 0.f;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int k = warp * 8 + 2 * t + e;
      const float w0 = expf(s[e] - n0), w1 = expf(s[2 + e] - n1);
      y0 += w0; y1 += w1;
      split_bf16(w0, m.Ph[g * PS + k], m.Pl[g * PS + k]);
      split_bf16(w1, m.Ph[(g + 8) * PS + k], m.Pl[(g + 8) * PS + k]);
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
      pfa_ldm4(ah, m.Ph + aoff);
      pfa_ldm4(al, m.Pl + aoff);
#pragma unroll
      for (int i = 0; i < TW / 2; ++i) {
        const int tile = 2 * (warp + LAS_WARPS * i);
        if (tile < tiles) {  // an odd last tile reads the row's next eight columns and drops them
          uint32_t vb[4];
          pfa_ldm4t(vb, m.Ks + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * RS + tile * 8 + (lane >> 4) * 8);
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
  if (t == 0) { st.sum[warp][g] = l0; st.sum[warp][g + 8] = l1; st.mx[warp][g] = m0; st.mx[warp][g + 8] = m1; }
  __syncthreads();
}

// Calls put(head, column, first, second) for the pairs of columns this thread holds after split_attend.
template <int TW, typename Put>
__device__ __forceinline__ void split_columns(const float (&o)[TW][4], int tiles, int nh, Put put) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int i = 0; i < TW; ++i) {
    const int tile = 2 * (warp + LAS_WARPS * (i >> 1)) + (i & 1);
    if (tile < tiles) {
      if (g < nh) put(g, 8 * tile + 2 * t, o[i][0], o[i][1]);
      if (g + 8 < nh) put(g + 8, 8 * tile + 2 * t, o[i][2], o[i][3]);
    }
  }
}

// ---- prompts -----------------------------------------------------------------------------------------------------
// 128 queries of one head per block over cached or expanded keys and values, 64-key tiles, online softmax, bfloat16
// tensor-core products (mma.sync m16n8k16) with FP32 scores and sums.
constexpr int LAP_Q = 128, LAP_K = 64, LAP_THREADS = 256, LAP_WARPS = 8;

// Query columns are E = dim + rot_dim wide; columns rot0 .. rot0 + rot_dim - 1 meet the separately stored rotated key parts,
// the others the columns of the same number of the key row. Keys lie in rows of a contiguous context (ring = 0: run.ctx0
// onwards), or in a slot's ring of `ring` rows (position p in row p % ring).
struct PromptAttnParams {
  const float* q;            // [T][q_stride], unrotated
  int q_stride;
  const float* rope;
  int pairs;
  const __nv_bfloat16* kv;   // [row][kv_stride]: key columns, the head's values from column v_off on
  int kv_stride, v_off;
  const __nv_bfloat16* kr;   // [row][kr_stride] rotated key parts
  int kr_stride;
  int group;                 // query heads per key / value head
  size_t k_head, v_head, kr_head;  // elements from one key / value head to the next in kv (keys, values) and kr
  int ring;
  size_t slot_elems;         // ring: elements from one slot to the next
  const float* gate;         // [T][gate_stride], or nullptr
  int gate_stride;
  const RunDesc* runs;
  int heads, dim, rot_dim, rot0, vdim;
  int wave;                  // blocks that start together, one per SM
  KeyMask mask;
  float scale, softcap;      // softcap: see capped_score
  int sink;                  // one more term exp(0) in the softmax denominator
  __nv_bfloat16* out;        // [T][out_stride]
  int out_stride;
};

__host__ __device__ __forceinline__ int lap_qk_stride(int dim, int rot) { return (dim + rot + 15) / 16 * 16 + 8; }
__host__ __device__ __forceinline__ int lap_value_cols(int vdim) { return vdim <= 32 ? 32 : vdim <= 64 ? 64 : vdim <= 128 ? 128 : 256; }
__host__ __device__ __forceinline__ size_t lap_smem_bytes(int dim, int rot, int vp) {
  return ((size_t)(LAP_Q + LAP_K) * lap_qk_stride(dim, rot) + (size_t)LAP_K * (vp + 8)) * 2;
}

// grid = (query blocks of the longest run * heads, 1, runs). VP = value columns per head rounded up to 32, 64, 128 or 256.
template <int VP>
__global__ void __launch_bounds__(LAP_THREADS, VP <= 128 ? 2 : 1) prompt_attn_kernel(const PromptAttnParams p) {
  extern __shared__ __align__(16) unsigned char lap_smem[];
  const RunDesc run = p.runs[blockIdx.z];
  // later queries may see more keys: the heaviest blocks come first, and every second wave of blocks runs through the order
  // backwards, so that blocks that share an SM add up to about the same
  int order = blockIdx.x;
  {
    const int wave = order / p.wave, first = wave * p.wave;
    if (wave & 1) order = first + min(p.wave, (int)gridDim.x - first) - 1 - (order - first);
  }
  const int q0 = (gridDim.x / p.heads - 1 - order / p.heads) * LAP_Q, h = order % p.heads;
  if (q0 >= run.len) return;
  const int E = p.dim + p.rot_dim, EP = (E + 15) / 16 * 16, QS = EP + 8;
  constexpr int VS = VP + 8, NT_O = VP / 8;
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(lap_smem);
  __nv_bfloat16* Ks = Qs + LAP_Q * QS;
  __nv_bfloat16* Vs = Ks + LAP_K * QS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int nq = min(LAP_Q, run.len - q0);
  const bool vec = !((E | p.rot0 | p.rot_dim | p.vdim | p.kv_stride | p.v_off | p.kr_stride | p.q_stride | (int)p.k_head | (int)p.v_head | (int)p.kr_head) & 7);
  const size_t slot_at = p.ring ? run.slot * p.slot_elems : 0;
  const __nv_bfloat16* keys = p.kv + slot_at + h / p.group * p.k_head;
  const __nv_bfloat16* values = p.kv + slot_at + h / p.group * p.v_head + p.v_off;
  const __nv_bfloat16* rotated_keys = p.kr + slot_at + h / p.group * p.kr_head;
  const int rot1 = p.rot0 + p.rot_dim;
  // queries, rotated; the scale is applied to the products
  if (vec) {  // pieces of four elements (two pairs), eight of them in flight per thread
    const int n4 = EP >> 2, d4 = p.rot0 >> 2, e4 = E >> 2;
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
        if (r < nq && c < E) v = c >= p.rot0 && c < rot1 ? rotated(qr + p.rot0, c - p.rot0, table, p.pairs) : qr[c];
        Qs[r * QS + c] = __float2bfloat16(v);
      }
    }
  }
  const int qpos0 = run.start + q0;                       // position of the block's first query
  const int kfirst = p.mask.first(qpos0), klast = qpos0 + nq - 1;
  const int my0 = qpos0 + warp * 16 + g, my1 = my0 + 8;   // this thread's two query positions
  float o[NT_O][4];
#pragma unroll
  for (int i = 0; i < NT_O; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  // a sink is a key of score 0 without a value: it is there from the start (sums are shared by the four lanes of a row)
  float m0 = p.sink ? 0.f : -INFINITY, m1 = m0, l0 = p.sink && t == 0 ? 1.f : 0.f, l1 = l0;
  constexpr float LOG2E = 1.4426950408889634f;
  const float sc2 = p.scale * LOG2E, cap2 = p.softcap * LOG2E, to_tanh = p.softcap > 0.f ? 2.f * LOG2E * p.scale / p.softcap : 0.f;
  const int wfirst = qpos0 + warp * 16, whigh = min(wfirst + 15, klast), wlow = p.mask.first(wfirst), wlast = p.mask.first(wfirst + 15);  // of the warp's queries
  const int base = run.start - run.hist;                  // contiguous context: position of its first row
  auto first_row = [&](int kt) { return p.ring ? kt % p.ring : run.ctx0 + kt - base; };
  auto row_of = [&](int row0, int r) { return p.ring && row0 + r >= p.ring ? row0 + r - p.ring : row0 + r; };  // r rows further
  // 16-byte pieces of a tile: a thread keeps its column and takes every k_rows-th (v_rows-th) row
  constexpr int CV = VP >> 3, V_ROWS = LAP_THREADS / CV;
  const int ce = EP >> 3, k_rows = LAP_THREADS / ce, kr0 = tid / ce, kc = tid - kr0 * ce;
  const bool k_rot = kc >= p.rot0 >> 3 && kc < rot1 >> 3, k_has = kc < E >> 3;
  const __nv_bfloat16* k_src = k_rot ? rotated_keys + 8 * kc - p.rot0 : keys + 8 * kc;
  const int k_ld = k_rot ? p.kr_stride : p.kv_stride;

  // Key and value tiles have one buffer each: the next key tile is requested as soon as this one's scores are done, the
  // next value tile after this one's products, so each copy runs under the other half of the work.
  auto load_k = [&](int kt) {
    const int nk = min(LAP_K, klast - kt + 1), row0 = first_row(kt);
    if (vec) {
      if (kr0 < k_rows)
        for (int r = kr0; r < LAP_K; r += k_rows) {
          __nv_bfloat16* d = Ks + r * QS + 8 * kc;
          if (r < nk && k_has) pfa_cp16(d, k_src + (size_t)row_of(row0, r) * k_ld);
          else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
        }
    } else {
      for (int i = tid; i < LAP_K * EP; i += LAP_THREADS) {
        const int r = i / EP, c = i - r * EP;
        __nv_bfloat16 v = __float2bfloat16(0.f);
        if (r < nk && c < E) {
          const size_t row = row_of(row0, r);
          v = c >= p.rot0 && c < rot1 ? rotated_keys[row * p.kr_stride + c - p.rot0] : keys[row * p.kv_stride + c];
        }
        Ks[r * QS + c] = v;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto load_v = [&](int kt) {
    const int nk = min(LAP_K, klast - kt + 1), row0 = first_row(kt);
    if (vec) {
      const int c = tid % CV;
      const bool has = c < p.vdim >> 3;
      const __nv_bfloat16* src = values + 8 * c;
#pragma unroll
      for (int i = 0; i < LAP_K / V_ROWS; ++i) {
        const int r = tid / CV + i * V_ROWS;
        __nv_bfloat16* d = Vs + r * VS + 8 * c;
        if (r < nk && has) pfa_cp16(d, src + (size_t)row_of(row0, r) * p.kv_stride);
        else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
      }
    } else {
      for (int i = tid; i < LAP_K * VP; i += LAP_THREADS) {
        const int r = i / VP, c = i - r * VP;
        Vs[r * VS + c] = r < nk && c < p.vdim ? values[(size_t)row_of(row0, r) * p.kv_stride + c] : __float2bfloat16(0.f);
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
    const bool sees = kt <= whigh && kt + LAP_K > wlow;  // some query of this warp sees some key of the tile
    float s[8][4];
    if (sees) {
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
    }
    __syncthreads();  // every warp has read the key tile
    if (kt + LAP_K <= klast) load_k(kt + LAP_K);
    else asm volatile("cp.async.commit_group;" ::: "memory");  // keeps one group per step
    if (sees) {
      if (p.softcap > 0.f) {  // cap * tanh(x / cap) with tanh(z) = 1 - 2 / (1 + e^(2z)), then to base 2
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[i][e] = fmaf(-2.f * cap2, rcp_fast(1.f + ex2_fast(s[i][e] * to_tanh)), cap2);
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[i][e] *= sc2;
      }
      if (kt + LAP_K - 1 > wfirst || kt < wlast) {  // not every query of the warp sees every key
        const int low0 = p.mask.first(my0), low1 = p.mask.first(my1);
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int key = kt + 8 * i + 2 * t + e;
            if (key > my0 || key < low0) s[i][e] = -INFINITY;
            if (key > my1 || key < low1) s[i][2 + e] = -INFINITY;
          }
      }
      float n0 = m0, n1 = m1;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        n0 = fmaxf(n0, fmaxf(s[i][0], s[i][1]));
        n1 = fmaxf(n1, fmaxf(s[i][2], s[i][3]));
      }
#pragma unroll
      for (int x = 1; x < 4; x <<= 1) {
        n0 = fmaxf(n0, __shfl_xor_sync(0xffffffffu, n0, x));
        n1 = fmaxf(n1, __shfl_xor_sync(0xffffffffu, n1, x));
      }
      // a row that has seen no key yet keeps -infinity: subtract 0 then, every weight is 2^-inf = 0
      const float z0 = n0 == -INFINITY ? 0.f : n0, z1 = n1 == -INFINITY ? 0.f : n1;
      if (__any_sync(0xffffffffu, n0 != m0 || n1 != m1)) {
        const float f0 = ex2_fast(m0 - z0), f1 = ex2_fast(m1 - z1);
        l0 *= f0; l1 *= f1;
#pragma unroll
        for (int i = 0; i < NT_O; ++i) { o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1; }
      }
      m0 = n0; m1 = n1;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          s[i][e] = ex2_fast(s[i][e] - z0);
          s[i][2 + e] = ex2_fast(s[i][2 + e] - z1);
          l0 += s[i][e];
          l1 += s[i][2 + e];
        }
      }
    }
    asm volatile("cp.async.wait_group 1;" ::: "memory");  // the value tile
    __syncthreads();
    // weighted values
    if (sees) {
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
        p.out[row * p.out_stride + j] = __float2bfloat16(o[i][e] * (e < 2 ? i0 : i1) * (p.gate ? p.gate[row * p.gate_stride + j] : 1.f));
      }
    }
  }
}

}  // namespace b200
