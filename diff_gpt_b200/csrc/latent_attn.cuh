// Arguments and key ranges shared by the kernels that attend to cached rows (latent_attn.cu, latent_tc.cu).
//
// A cache holds one row of `row_w` numbers per token.  Query head h belongs to group g = h / (H / G); the group's key is
// columns [g dk, +dk) of a row and its value columns [v_col + g dv, +dv).  Attention on latents is the case of one group
// whose value is its key (dk = dv, v_col = 0); grouped-query attention stores the G keys and then the G values.
#pragma once

#include "common.cuh"

namespace dgpt {

struct LatentArgs {
  const void* q;
  long long q_rs;
  KvView kv;
  const int* len0;
  const int* start1;
  const int* len1;
  const int* step_ptr;
  const void* gate;
  long long gate_rs;
  void* out;
  long long out_rs;
  float* ws_o;
  float* ws_ml;
  int n_splits, n_seq, Tn, H, window;
  int G, dk, dv;    // groups, query / key size, value size
  int row_w, v_col; // elements between rows; where the values start
  int keep;         // the first `keep` keys are seen from every distance
  float scale_log2;
  int* status;
};

// The keys of one query row: logical keys [0, ks) and [lo, n); key i is slot i below n0 and slot s1 + (i - n0) from there on.
struct LatentKeys {
  int seq, n0, s1, ks, lo, n;
};
__device__ __forceinline__ LatentKeys latent_keys(const LatentArgs& a, int row) {
  LatentKeys k;
  k.seq = row / a.Tn;
  const int t = row - k.seq * a.Tn;
  const int cap = a.kv.page_table ? a.kv.max_pages * a.kv.page_tokens : a.kv.page_tokens;
  k.n0 = a.len0 ? min(max(a.len0[k.seq], 0), cap) : 0;
  k.s1 = min(max(a.start1[k.seq], 0), cap);
  const int n1 = a.len1[k.seq] + (a.step_ptr ? *a.step_ptr : 0) + t;
  k.n = k.n0 + min(max(n1, 0), cap - k.s1);  // never past the sequence's slots
  k.lo = a.window > 0 ? max(0, k.n - a.window) : 0;
  k.ks = min(a.keep, k.lo);
  return k;
}

// tcgen05 form (latent_tc.cu): bf16, dk, dv <= 512, dense runs or pages that tile its 128-key blocks
bool latent_tc_supported(const LatentArgs& a, const dgpt_kv_layout& kv, int dtype);
int latent_tc_launch(const LatentArgs& a, const dgpt_kv_layout& kv, cudaStream_t st);

}  // namespace dgpt
