// stack_pool.cuh — attention with pooled blocks behind its window and mixed heads (stack_pool.cu): the per-token preparation of
// q | k | v (short causal convolution, per-head norms, rotary positions of either pair layout) straight into the caches, the block
// means, and the attention itself.  Storage type T = bf16 or fp32; convolutions, norms, angles, scores, the softmax and the mixing of
// its weights are fp32.
//
// The key list of a query at position i is [blocks 0 … nb − 1 | tokens lo … i]: lo = max(0, i − window + 1), and nb = the
// blocks of `pool` positions that end before the window, floor((i − window + 1) / pool).  The caches of a run hold max_ctx token
// rows and behind them max_ctx / pool block rows; block b is written when its last token is, so it is complete before any
// position that sees it.  (The preparation, launch_pool_prep, also serves the plain attention of sandwich blocks.)
#pragma once
#include "stack.cuh"

namespace b200 {

constexpr int kPoolMaxSplits = 64;
constexpr int kPoolTile = 32;          // keys per tile of the general kernels

struct PoolAttn {
  b200_attn_desc a{};
  b200_pool_attn_desc d{};
  float eps = 1e-5f;
  const void* proj = nullptr;    // [n_tok, ld_proj] T: q | k | v at off_q / off_k / off_v, biases included
  int64_t ld_proj = 0;
  int off_q = 0, off_k = 0, off_v = 0;
  void* q = nullptr;             // [n_tok, heads·dim] T: prepared queries
  void* kcache = nullptr;        // this run's rows of slot 0; slot s is s·k_slot_stride elements further
  void* vcache = nullptr;
  int64_t k_slot_stride = 0, v_slot_stride = 0;
  int max_ctx = 0;
  float* conv_state = nullptr;   // slot 0's [taps − 1][ld_proj] fp32
  int64_t conv_slot_stride = 0;
  int q_only = 0;                // 1: the rows hold queries only (a layer that reads another layer's cached keys and values)
  int heads_per_cta = 0;         // launch_pool_prep: query heads one CTA prepares (set by the launcher)
  int single = 0;                // 1: every row is its sequence's only new one — the preparation moves the convolution's state
                                 // on and pools a finished block itself
  const int32_t* slot = nullptr;
  const int32_t* pos = nullptr;
  int n_tok = 0;
  // the step's sequences (launch_pool_blocks): first row and row count of each, the most rows any of them brings
  const int32_t *seg_row0 = nullptr, *seg_count = nullptr;
  int n_seg = 0, max_count = 0;
  // attention workspaces: scores [n_tok][heads][nk_max], softmax parts [n_tok][heads][nsplit][2], outputs
  // [n_tok][nsplit][heads·vdim] (nsplit > 1), all fp32; nk_max >= every row's key list, nsplit · keys_per_split >= nk_max
  float *scores = nullptr, *parts = nullptr, *outs = nullptr;
  int nk_max = 0, nsplit = 1, keys_per_split = 0;
  void* mid = nullptr;           // [n_tok, ld_mid] T: head h at columns h·vdim, columns [heads·vdim, n_pad) get zeros
  int64_t ld_mid = 0;
  int n_pad = 0;
  float out_scale = 1.f;
};
// block rows a run's cache holds behind its token rows
__host__ __device__ inline int pool_rows(int max_ctx, int pool) { return pool > 0 ? max_ctx / pool : 0; }
// most keys a query sees in a cache of `ctx` positions
inline int pool_keys_max(int ctx, int window, int pool) {
  if (window <= 0 || window >= ctx) return ctx;
  return window + (pool > 0 ? (ctx - window) / pool : 0);
}
int launch_pool_prep(const PoolAttn& p, int dtype, cudaStream_t st);      // queries, cache rows, (single: blocks, state)
int launch_pool_blocks(const PoolAttn& p, int dtype, cudaStream_t st);    // the blocks that end in this step's rows
int launch_pool_attention(const PoolAttn& p, int dtype, cudaStream_t st); // any shape
// bf16 prompts on the tensor cores (stack_pool_mma.cu): the sequences [seg_row0, + seg_count) of the step (device arrays) that bring
// min_rows rows or more, max_count the most any of them brings; stats: fp32 [n_tok][heads][2].  pool_prompt_ok: head sizes that
// are multiples of 16 (dim <= 128, vdim <= 256), up to 32 heads, and the queries and one key / value tile of all heads fit one
// CTA's shared memory.
bool pool_prompt_ok(const b200_attn_desc& a);
int launch_pool_prompt(const PoolAttn& p, const int32_t* seg_row0, const int32_t* seg_count, int n_seg, int max_count, int min_rows,
                       float* stats, cudaStream_t st);

#ifdef __CUDACC__
__device__ __forceinline__ int pool_lo(int i, int window) { return window > 0 ? max(0, i - window + 1) : 0; }
__device__ __forceinline__ int pool_nb(int i, int window, int pool) {
  return window > 0 && pool > 0 && i - window + 1 > 0 ? (i - window + 1) / pool : 0;
}
#endif

}  // namespace b200
