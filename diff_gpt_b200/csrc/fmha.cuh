// Argument block shared by the two prefill-attention kernels.
#pragma once

#include "common.cuh"

namespace dgpt {

struct FmhaArgs {
  const void* q;
  long long q_bs, q_rs;
  const int* kv_len;
  int kv_len_all;
  void* o;
  long long o_bs, o_rs;
  int o_f32;
  float* lse;
  int B, H, Tq, D, q_offset, causal, dtype;
  int* status;
  int max_ctas;  // two-CTAs-per-SM kernel only: at most this many CTAs, looping over the query tiles (0 = one CTA per tile)
  int two_cta;  // tensor-core path only: the 128-thread kernel with two CTAs per SM instead of the warp-specialised one
  int pingpong;  // tensor-core path only: the kernel with two query tiles per CTA
  // sliding-window form (dgpt_fmha_window); the defaults leave the kernels as dgpt_fmha_prefill uses them
  int window = 0;           // query i sees keys (q_offset + i - window, q_offset + i]; 0 = all of them (causal only)
  float scale = 0.f;        // score scale; 0 = 1 / sqrt(D)
  long long kv_ts = 0;      // elements between consecutive keys of a head; 0 = D
  int kv_heads = 0;         // key/value heads; query head h reads h / (H / kv_heads); 0 = H
  int keep_first = 0;       // with a window: keys j < keep_first are seen from every distance
  const void* hgate = nullptr;  // [B * Tq, H] in dtype: output of head h is multiplied by sigmoid(hgate)
  long long hgate_rs = 0;
};

// What the tensor-core kernels need besides the three tensor maps.
struct TcParams {
  const int* kv_len;
  int kv_len_all;
  const int* page_table;
  int max_pages;
  int page_tokens;
  void* o;
  long long o_bs, o_rs;
  int o_f32;
  float* lse;
  int H, Tq, q_offset, causal;
  float scale_log2;
  int* status;
  int n_qt, n_work;  // query tiles per (batch, head) and work items in all (a capped grid loops over them)
  int d_head;        // head_dim of the tensors in global memory (32 rides on the 64-wide kernels: the TMA boxes are 64 wide
                     // and the columns past the tensor's extent arrive as zeros, so scores and outputs are unchanged)
  int window;        // 0 = no lower bound
  int keep_first;    // keys below this are seen whatever the window
  int kv_div;        // query heads per key/value head
  const void* hgate; // bf16 [B * Tq, H], or NULL
  long long hgate_rs;
  int BH, group_bh;  // two-query-tile kernel: (batch, head) pairs in all, and how many are worked on at a time
};

// Factor that the per-head output gate puts on row `row` (b * Tq + i) of head h.
template <typename T>
__device__ __forceinline__ float head_gate(const void* hgate, long long rs, long long row, int h) {
  if (hgate == nullptr) return 1.f;
  return 1.f / (1.f + expf(-Io<T>::ld(static_cast<const T*>(hgate) + row * rs + h)));
}
// First key tile of `tile` keys inside the window of a query at position `first_q` (the query tile's lowest).
__device__ __forceinline__ int window_first_tile(int window, int first_q, int tile) {
  return window > 0 ? max(0, first_q - window + 1) / tile : 0;
}
// Key tiles ahead of that one that hold kept first keys.  A query tile visits the n_window tiles from `tile0` on and then
// tiles [0, n_kept): its j-th tile is tile_of(j).  (The kept ones last: by then the running maximum is settled, and a tile of
// which a few keys are seen seldom moves it.)
__device__ __forceinline__ int kept_tiles(int keep_first, int tile0, int tile) {
  return min(tile0, (keep_first + tile - 1) / tile);
}
template <bool KEPT>
__device__ __forceinline__ int tile_of(int j, int n_window, int tile0) {
  return KEPT && j >= n_window ? j - n_window : tile0 + j;
}

// warp-level kernel (fmha_simt.cu)
int fmha_simt(const FmhaArgs& a, const KvView& kv, cudaStream_t st);

// tcgen05 / TMEM kernel (fmha_tc.cu)
bool fmha_tc_supported(const FmhaArgs& a, const dgpt_kv_layout& kv);
int fmha_tc(const FmhaArgs& a, const dgpt_kv_layout& kv, cudaStream_t st);
// the same with two query tiles per CTA taking turns on the tensor cores (fmha_pp.cu); `tp` and the maps come from fmha_tc
struct TcMaps;
int fmha_tc_pp_launch(const FmhaArgs& a, const TcMaps& maps, TcParams p, long long kv_span, cudaStream_t st);
// the persistent warp-specialised kernel with one query tile per work item (fmha_ws.cu)
int fmha_tc_ws_launch(const FmhaArgs& a, const TcMaps& maps, TcParams p, long long kv_span, cudaStream_t st);

}  // namespace dgpt
