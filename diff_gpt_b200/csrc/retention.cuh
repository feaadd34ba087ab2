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

}  // namespace dgpt
