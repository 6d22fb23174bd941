// Device-resident state of a block model (model_registry.h): weights, the per-run caches and recurrent states of every
// sequence slot, and the buffers of the decode step and of a prompt chunk.
#pragma once
#include <cuda_bf16.h>

#include <vector>

#include "model_registry.h"

namespace b200 {

struct DenseW {
  __nv_bfloat16* w = nullptr;  // [rows][ld], ld = cols rounded up to a multiple of 8, zero-filled
  int rows = 0, cols = 0;
};

struct BlockLayer {
  // FP32 vectors, zero-filled up to a multiple of 8 elements
  float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
  DenseW o, gate_up /* interleaved by 8 rows */, down;
  // latent attention
  DenseW dq, dkv, g, uq, ukv /* W_uk rows, then W_uv rows */;
  float *dq_norm = nullptr, *dkv_norm = nullptr;
  const float* rope = nullptr;  // [max_ctx][rot.dims / 2]{cos, sin}, shared by layers with the same rotation
  // wkv
  DenseW r, k, v, wg, w1, w2;
  float *mu[5] = {nullptr}, *w0 = nullptr, *u = nullptr, *norm = nullptr;
  // shared-kv attention (keys: k)
  DenseW q;
  // rg-lru: the two branches, the gate matrices as [width][block size], the convolution as [taps][padded width]
  DenseW in_y, in_x, ra, ri;
  float *y_b = nullptr, *x_b = nullptr, *ra_b = nullptr, *ri_b = nullptr, *conv = nullptr, *conv_b = nullptr, *decay = nullptr;
};

// What one layer run keeps per sequence slot (a looped layer has one of these per pass).
struct BlockRun {
  int layer = 0;
  bool add_embedding = false;  // the embedding output joins the stream ahead of this run
  void* cache = nullptr;   // latent attention: ring of rows [slot][cap][crow]; shared-kv attention: [slot][kv_heads][cap][crow]
  int cap = 0, crow = 0, kvp = 0;
  size_t cache_slot_bytes = 0;
  float* state = nullptr;  // wkv: [slot][heads][dim][dim]; rg-lru: [slot][padded width]
  float* shift = nullptr;  // wkv: [slot][2][padded model width], the previous token's input by position parity; rg-lru: [slot][taps][padded width], the convolution's last inputs
  size_t state_slot = 0, shift_slot = 0;  // floats per slot
};

struct BlockModel {
  BlockSpec spec;
  bool f32 = false;
  std::vector<int> order;  // layer of every run
  std::vector<BlockLayer> layers;
  std::vector<BlockRun> runs;
  DenseW embed, head;      // head: the embedding table itself when they are tied
  float* first = nullptr;  // embedding output of the rows in work, kept for a loop that adds it again
  float* final_norm = nullptr;
  int Wp = 0;              // padded width
  int chunk = 1024;        // prompt tokens per chunk
  int rows_cap = 0;        // rows the buffers below hold
  std::vector<int> slot_len;  // tokens each slot holds: recurrent state and rings only continue where they stand
  int64_t step_launches = 0, step_weight_bytes = 0, kv_bytes_per_pos = 0;
  // decode step (matvec path), [max_seqs] rows
  float *y = nullptr, *cat = nullptr, *q = nullptr, *att = nullptr, *act = nullptr;
  int cat_stride = 0, q_stride = 0, att_stride = 0, act_stride = 0;
  float *part_o = nullptr, *part_ml = nullptr;
  int* tickets = nullptr;
  __nv_bfloat16* q_split[2] = {nullptr, nullptr};  // absorbed queries of decode attention: value and remainder, [max_seqs][heads][cache row]
  // row path: prompt chunks and batches of 16 and more, [rows_cap] rows
  float *rx = nullptr, *ry = nullptr, *rh = nullptr, *rcat = nullptr, *rq = nullptr, *rdecay = nullptr, *ro = nullptr;
  void *ra[5] = {nullptr};      // operand rows of the next matmul (five for token-shift mixes)
  void *ratt = nullptr, *ract = nullptr;
  int ra_stride = 0, decay_stride = 0;
  int* meta = nullptr;          // tokens | positions | slots | run tables | gather rows
  size_t meta_cap = 0;
  void *ctx = nullptr, *ctx_kr = nullptr, *ctx_kv = nullptr;  // expanded context of a chunk
  size_t ctx_cap[3] = {0, 0, 0};
  // split-K workspace of the tensor-core matmul
  float* gemm_ws = nullptr;
  size_t gemm_ws_floats = 0;
  int* gemm_tickets = nullptr;
  int gemm_tickets_cap = 0;
  float* logits = nullptr;      // [rows][vocab] of the wanted places, grown on demand
  size_t logits_cap = 0;
};

}  // namespace b200
