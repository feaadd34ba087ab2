// Arguments and key ranges shared by the latent-attention kernels (latent_attn.cu, latent_tc.cu).
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
  int n_splits, n_seq, Tn, H, r, window;
  float scale_log2;
  int* status;
};

// The keys of one row: logical keys [lo, n); key i is slot i below n0 and slot s1 + (i - n0) from there on.
struct LatentKeys {
  int seq, n0, s1, lo, n;
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
  return k;
}

// tcgen05 form (latent_tc.cu): bf16, r <= 512, dense runs or pages that tile its 128-key blocks
bool latent_tc_supported(const LatentArgs& a, const dgpt_kv_layout& kv, int dtype);
int latent_tc_launch(const LatentArgs& a, const dgpt_kv_layout& kv, cudaStream_t st);

}  // namespace dgpt
