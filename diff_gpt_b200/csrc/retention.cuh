// Arguments shared by the retention kernels (retention.cu, retention_tc.cu).
#pragma once

#include "common.cuh"

namespace dgpt {

struct RetentionArgs {
  const void* in;  // [n_seq * Tn, in_rs]: q, k, v and gate of all heads from these columns on
  long long in_rs;
  int q_col, k_col, v_col, g_col;
  const float2* table;  // [table_len, rot / 2] (cos, sin) per position
  int table_len, rot;
  const int* pos0;      // position of each sequence's first token, plus *step_ptr
  const int* step_ptr;
  const float* decay;   // [H]
  float k_scale;
  const float* state_in;  // [n_seq, H, dim, vdim], or NULL (zeros)
  float* state_out;       // the same after the call, or NULL
  float eps;
  void* y;  // [n_seq * Tn, H * vdim]
  long long y_rs;
  float* o;  // workspace
  int n_seq, Tn, H, dim, vdim, dim_pad;
  int* status;
};

// chunked form (retention_tc.cu): bf16, dim <= 128, decays (the smallest: min_decay) that leave a chunk room.  With several
// slices of value columns it leaves o in a.o, unnormalised; otherwise y is written.
bool retention_tc_supported(const RetentionArgs& a, int dtype, float min_decay);
size_t retention_tc_workspace_bytes(int n_seq, int T, int H, int dim, int vdim);
int retention_tc_launch(const RetentionArgs& a, float* seg_state, cudaStream_t st);

}  // namespace dgpt
