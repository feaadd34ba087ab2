// Row-wise kernels of models that keep their residual stream in fp32 and average it over depth:
//
//   embed_scale      X_0 = scale * Emb[ids]
//   norm_add         x' = x + rms_norm(y) * w                        (norm on a sublayer's output), and x' in the model dtype
//   depth_avg_conv   x = sum_j a_j X_j ;  h = x + causal_conv(x)      (h is what the next mixer reads)
//   layer_tail       the two above in one pass for one new token per sequence (decode)
//   depth_avg_norm   x = sum_j a_j X_j ;  out = rms_norm(x) * w        (in front of the output head)
//   xielu, silu_mul  activations, element-wise (the GEMM of gemm_tc.cu has them as epilogues)
//
// X_j are the fp32 [n, C] slices of one slab, `term_stride` elements apart; everything is accumulated in fp32.
// All of them are HBM-bound: each X_j row is read once and each output row written once.  VEC = 4 channels per thread
// where C is a multiple of 4, 1 otherwise.
#include "activation.cuh"
#include "rowvec.cuh"

namespace dgpt {

constexpr int kMaxTaps = 16;

// sum_j coef[j] * slab[j][off .. off + VEC)
template <int VEC>
__device__ __forceinline__ FVec<VEC> depth_sum(const float* __restrict__ slab, long long term_stride, int terms,
                                               const float* __restrict__ coef, long long off) {
  FVec<VEC> acc;
#pragma unroll
  for (int x = 0; x < VEC; ++x) acc.v[x] = 0.f;
  int j = 0;
  for (; j + 4 <= terms; j += 4) {  // four independent loads in flight
    FVec<VEC> t[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) t[u] = ldf<VEC>(slab + (long long)(j + u) * term_stride + off);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const float a = __ldg(coef + j + u);
#pragma unroll
      for (int x = 0; x < VEC; ++x) acc.v[x] += a * t[u].v[x];
    }
  }
  for (; j < terms; ++j) {
    const FVec<VEC> t = ldf<VEC>(slab + (long long)j * term_stride + off);
    const float a = __ldg(coef + j);
#pragma unroll
    for (int x = 0; x < VEC; ++x) acc.v[x] += a * t.v[x];
  }
  return acc;
}

// ---- X_0 ---------------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void embed_scale_kernel(const int* __restrict__ ids, const T* __restrict__ emb, float* __restrict__ out,
                                   long long n, int C, int V, float scale) {
  const int cv = C / VEC;
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n * cv) return;
  const long long row = i / cv;
  const int c = (int)(i - row * cv) * VEC;
  int id = ids[row];
  id = id < 0 ? 0 : (id >= V ? V - 1 : id);
  FVec<VEC> t = ldt<T, VEC>(emb + (long long)id * C + c);
#pragma unroll
  for (int x = 0; x < VEC; ++x) t.v[x] *= scale;
  stf<VEC>(out + row * C + c, t);
}

// ---- x + rms_norm(y) * w -------------------------------------------------------------------
// One CTA per row; NV vectors of the row per thread stay in registers between the two passes.
template <typename T, int VEC, int NV>
__global__ void __launch_bounds__(kRowThreads)
norm_add_kernel(const T* __restrict__ y, const float* __restrict__ w, float eps, const float* x, float* out, T* __restrict__ u,
                int C) {
  __shared__ float scratch[40];
  const long long row = blockIdx.x;
  const int cv = C / VEC;
  FVec<VEC> r[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = threadIdx.x + i * blockDim.x;
    if (j < cv) {
      r[i] = ldt<T, VEC>(y + row * C + j * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += r[i].v[e] * r[i].v[e];
    }
  }
  const float inv = rsqrtf(block_sum(ss, scratch) / (float)C + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = threadIdx.x + i * blockDim.x;
    if (j < cv) {
      const FVec<VEC> wv = ldf<VEC>(w + j * VEC);
      FVec<VEC> xv = ldf<VEC>(x + row * C + j * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) xv.v[e] += r[i].v[e] * inv * wv.v[e];
      stf<VEC>(out + row * C + j * VEC, xv);
      if (u) stt<T, VEC>(u + row * C + j * VEC, xv);
    }
  }
}

// ---- depth average, then h = x + conv(x) ------------------------------------------------------
// A thread owns VEC channels of a run of `seg` consecutive tokens of one sequence and keeps the last TAPS - 1 averaged
// values in registers; the tokens just before its run are averaged again (they were written by nobody yet), the ones
// before the call come from the sequence's state.  TAPS >= taps: a shorter filter sits at the end of the array.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(128)
depth_avg_conv_kernel(const float* __restrict__ slab, long long term_stride, int terms, const float* __restrict__ coef,
                      const float* __restrict__ cw, int taps, const float* state_in, float* state_out, float* x_out,
                      T* __restrict__ h_out, int n_seq, int Tn, int seg, int n_seg, int C) {
  const int cv = C / VEC;
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)n_seq * n_seg * cv) return;
  const int c = (int)(i % cv) * VEC;
  const int s = (int)((i / cv) % n_seg);
  const int b = (int)(i / ((long long)cv * n_seg));
  const int t_begin = s * seg, t_end = min(Tn, t_begin + seg);
  constexpr int HN = TAPS > 1 ? TAPS - 1 : 1;
  const int skip = TAPS - taps;  // unused entries at the front
  FVec<VEC> hist[HN], w[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    if (j >= skip) w[j] = ldf<VEC>(cw + (long long)(j - skip) * C + c);
    else {
#pragma unroll
      for (int x = 0; x < VEC; ++x) w[j].v[x] = 0.f;
    }
  }
  const long long row0 = (long long)b * Tn;
  const long long st0 = (long long)b * (taps - 1) * C + c;
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int t = t_begin - (TAPS - 1) + j;
#pragma unroll
    for (int x = 0; x < VEC; ++x) hist[j].v[x] = 0.f;
    if (j < skip) continue;
    if (t >= 0) hist[j] = depth_sum<VEC>(slab, term_stride, terms, coef, (row0 + t) * C + c);
    else if (state_in) hist[j] = ldf<VEC>(state_in + st0 + (long long)(t + taps - 1) * C);
  }
  for (int t = t_begin; t < t_end; ++t) {
    const long long off = (row0 + t) * C + c;
    const FVec<VEC> xv = depth_sum<VEC>(slab, term_stride, terms, coef, off);
    if (x_out) stf<VEC>(x_out + off, xv);
    FVec<VEC> h;
#pragma unroll
    for (int x = 0; x < VEC; ++x) h.v[x] = w[TAPS - 1].v[x] * xv.v[x];
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
#pragma unroll
      for (int x = 0; x < VEC; ++x) h.v[x] += w[j].v[x] * hist[j].v[x];
    }
#pragma unroll
    for (int x = 0; x < VEC; ++x) h.v[x] += xv.v[x];
    stt<T, VEC>(h_out + off, h);
#pragma unroll
    for (int j = 0; j + 1 < TAPS - 1; ++j) hist[j] = hist[j + 1];
    if (TAPS > 1) hist[HN - 1] = xv;
  }
  if (state_out && t_end == Tn) {
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j)
      if (j >= skip) stf<VEC>(state_out + st0 + (long long)(j - skip) * C, hist[j]);
  }
}

// ---- one new token per sequence: norm_add, depth average and convolution in one pass ------------
// CTA per row.  The new X (slab term terms - 1) is formed here from x1 and y and also written there; the state is
// shifted in place (each thread owns its channels).
template <typename T, int VEC, int NV>
__global__ void __launch_bounds__(kRowThreads)
layer_tail_kernel(const T* __restrict__ y, const float* __restrict__ nw, float eps, const float* __restrict__ x1, float* slab,
                  long long term_stride, int terms, const float* __restrict__ coef, const float* __restrict__ cw, int taps,
                  float* state, float* __restrict__ x_out, T* __restrict__ h_out, int C) {
  __shared__ float scratch[40];
  const long long row = blockIdx.x;
  const int cv = C / VEC;
  FVec<VEC> r[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = threadIdx.x + i * blockDim.x;
    if (j < cv) {
      r[i] = ldt<T, VEC>(y + row * C + j * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += r[i].v[e] * r[i].v[e];
    }
  }
  const float inv = rsqrtf(block_sum(ss, scratch) / (float)C + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = threadIdx.x + i * blockDim.x;
    if (j >= cv) continue;
    const int c = j * VEC;
    const long long off = row * C + c;
    const FVec<VEC> wv = ldf<VEC>(nw + c);
    FVec<VEC> xn = ldf<VEC>(x1 + off);
#pragma unroll
    for (int e = 0; e < VEC; ++e) xn.v[e] += r[i].v[e] * inv * wv.v[e];
    stf<VEC>(slab + (long long)(terms - 1) * term_stride + off, xn);
    FVec<VEC> xv = depth_sum<VEC>(slab, term_stride, terms - 1, coef, off);
    const float last = __ldg(coef + terms - 1);
#pragma unroll
    for (int e = 0; e < VEC; ++e) xv.v[e] += last * xn.v[e];
    stf<VEC>(x_out + off, xv);
    const FVec<VEC> w0 = ldf<VEC>(cw + (long long)(taps - 1) * C + c);
    FVec<VEC> h;
#pragma unroll
    for (int e = 0; e < VEC; ++e) h.v[e] = w0.v[e] * xv.v[e];
    float* st = state + row * (taps - 1) * C + c;
    for (int k = 0; k < taps - 1; ++k) {
      const FVec<VEC> sv = ldf<VEC>(st + (long long)k * C), wk = ldf<VEC>(cw + (long long)k * C + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) h.v[e] += wk.v[e] * sv.v[e];
      if (k > 0) stf<VEC>(st + (long long)(k - 1) * C, sv);
    }
    if (taps > 1) stf<VEC>(st + (long long)(taps - 2) * C, xv);
#pragma unroll
    for (int e = 0; e < VEC; ++e) h.v[e] += xv.v[e];
    stt<T, VEC>(h_out + off, h);
  }
}

// ---- depth average and the norm in front of the head -----------------------------------------
template <typename T, int VEC, int NV>
__global__ void __launch_bounds__(kRowThreads)
depth_avg_norm_kernel(const float* __restrict__ slab, long long term_stride, int terms, const float* __restrict__ coef,
                      const float* __restrict__ w, float eps, const int* __restrict__ row_index, T* __restrict__ out,
                      long long n, int C) {
  __shared__ float scratch[40];
  const long long row = blockIdx.x;
  long long src = row_index ? (long long)row_index[row] : row;
  src = src < 0 ? 0 : (src >= n ? n - 1 : src);
  const int cv = C / VEC;
  FVec<VEC> r[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = threadIdx.x + i * blockDim.x;
    if (j < cv) {
      r[i] = depth_sum<VEC>(slab, term_stride, terms, coef, src * C + j * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += r[i].v[e] * r[i].v[e];
    }
  }
  const float inv = rsqrtf(block_sum(ss, scratch) / (float)C + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = threadIdx.x + i * blockDim.x;
    if (j < cv) {
      const FVec<VEC> wv = ldf<VEC>(w + j * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) r[i].v[e] *= inv * wv.v[e];
      stt<T, VEC>(out + row * C + j * VEC, r[i]);
    }
  }
}

template <typename T, int VEC>
__global__ void xielu_kernel(const T* __restrict__ in, T* __restrict__ out, long long n, float alpha_p, float alpha_n) {
  const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (i >= n) return;
  FVec<VEC> t = ldt<T, VEC>(in + i);
#pragma unroll
  for (int x = 0; x < VEC; ++x) t.v[x] = xielu_value(t.v[x], alpha_p, alpha_n);
  stt<T, VEC>(out + i, t);
}

// out[i] = silu(in[2 i]) * in[2 i + 1]: gate and up columns interleaved
template <typename T, int VEC>
__global__ void silu_mul_kernel(const T* __restrict__ in, T* __restrict__ out, long long n_out) {
  const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (i >= n_out) return;
  FVec<VEC> a, b, r;
  if constexpr (VEC == 4) {
    a = ldt<T, VEC>(in + 2 * i);
    b = ldt<T, VEC>(in + 2 * i + 4);
    r.v[0] = silu_mul_value(a.v[0], a.v[1]);
    r.v[1] = silu_mul_value(a.v[2], a.v[3]);
    r.v[2] = silu_mul_value(b.v[0], b.v[1]);
    r.v[3] = silu_mul_value(b.v[2], b.v[3]);
  } else {
    r.v[0] = silu_mul_value(Io<T>::ld(in + 2 * i), Io<T>::ld(in + 2 * i + 1));
  }
  stt<T, VEC>(out + i, r);
}

}  // namespace dgpt

using namespace dgpt;

#define DGPT_ROW_DISPATCH(KERNEL, TT, VV, ...)                                                                     \
  do {                                                                                                             \
    const int cv_ = C / VV, th_ = row_threads(cv_), nv_ = (cv_ + th_ - 1) / th_;                                   \
    if (nv_ <= 1) KERNEL<TT, VV, 1><<<(unsigned)rows_, th_, 0, st>>>(__VA_ARGS__);                                 \
    else if (nv_ <= 2) KERNEL<TT, VV, 2><<<(unsigned)rows_, th_, 0, st>>>(__VA_ARGS__);                            \
    else if (nv_ <= 4) KERNEL<TT, VV, 4><<<(unsigned)rows_, th_, 0, st>>>(__VA_ARGS__);                            \
    else if (nv_ <= 8) KERNEL<TT, VV, 8><<<(unsigned)rows_, th_, 0, st>>>(__VA_ARGS__);                            \
    else if (nv_ <= 16) KERNEL<TT, VV, 16><<<(unsigned)rows_, th_, 0, st>>>(__VA_ARGS__);                          \
    else {                                                                                                         \
      set_error(#KERNEL ": width %d is not built", C);                                                             \
      return DGPT_E_UNSUPPORTED;                                                                                   \
    }                                                                                                              \
  } while (0)

extern "C" int dgpt_embed_scale(const int32_t* ids, const void* emb, float* out, int64_t n_tokens, int32_t C, int32_t V,
                                float scale, int32_t dtype, void* stream) {
  DGPT_REQUIRE(ids && emb && out, "embed_scale: NULL pointer");
  DGPT_REQUIRE(n_tokens >= 0 && C > 0 && V > 0, "embed_scale: bad sizes");
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, "embed_scale: unknown dtype %d", dtype);
  if (n_tokens == 0) return DGPT_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool v4 = C % 4 == 0 && al16(emb) && al16(out);
  const long long work = (long long)n_tokens * (v4 ? C / 4 : C);
  const unsigned grid = (unsigned)((work + 255) / 256);
  const float* ef = static_cast<const float*>(emb);
  const __nv_bfloat16* eb = static_cast<const __nv_bfloat16*>(emb);
  if (dtype == DGPT_F32) {
    if (v4) embed_scale_kernel<float, 4><<<grid, 256, 0, st>>>(ids, ef, out, n_tokens, C, V, scale);
    else embed_scale_kernel<float, 1><<<grid, 256, 0, st>>>(ids, ef, out, n_tokens, C, V, scale);
  } else {
    if (v4) embed_scale_kernel<__nv_bfloat16, 4><<<grid, 256, 0, st>>>(ids, eb, out, n_tokens, C, V, scale);
    else embed_scale_kernel<__nv_bfloat16, 1><<<grid, 256, 0, st>>>(ids, eb, out, n_tokens, C, V, scale);
  }
  return launch_status("embed_scale");
}

extern "C" int dgpt_norm_add(const void* y, const float* w, float eps, const float* x, float* out, void* u, int64_t rows,
                             int32_t C, int32_t dtype, void* stream) {
  DGPT_REQUIRE(y && w && x && out, "norm_add: NULL pointer");
  DGPT_REQUIRE(rows >= 0 && rows <= 0x7fffffff && C > 0, "norm_add: bad sizes");
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, "norm_add: unknown dtype %d", dtype);
  if (rows == 0) return DGPT_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const long long rows_ = rows;
  const bool v4 = C % 4 == 0 && al16(y) && al16(w) && al16(x) && al16(out) && al16(u);
#define DGPT_NA(TT, VV) \
  DGPT_ROW_DISPATCH(norm_add_kernel, TT, VV, static_cast<const TT*>(y), w, eps, x, out, static_cast<TT*>(u), C)
  if (dtype == DGPT_F32) {
    if (v4) DGPT_NA(float, 4);
    else DGPT_NA(float, 1);
  } else {
    if (v4) DGPT_NA(__nv_bfloat16, 4);
    else DGPT_NA(__nv_bfloat16, 1);
  }
#undef DGPT_NA
  return launch_status("norm_add");
}

extern "C" int dgpt_depth_avg_conv(const float* slab, int64_t term_stride, int32_t terms, const float* coef,
                                   const float* conv_w, int32_t taps, const float* state_in, float* state_out, float* x_out,
                                   void* h_out, int32_t n_seq, int32_t T, int32_t C, int32_t dtype, void* stream) {
  DGPT_REQUIRE(slab && coef && conv_w && h_out, "depth_avg_conv: NULL pointer");
  DGPT_REQUIRE(terms >= 1 && n_seq >= 0 && T >= 0 && C > 0, "depth_avg_conv: bad sizes");
  DGPT_REQUIRE(taps >= 1 && taps <= kMaxTaps, "depth_avg_conv: taps must be in [1, %d]", kMaxTaps);
  DGPT_REQUIRE(state_in == nullptr || state_in != state_out || T <= 1,
               "depth_avg_conv: the state may be updated in place for T = 1 only");
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, "depth_avg_conv: unknown dtype %d", dtype);
  if (n_seq == 0 || T == 0) return DGPT_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool v4 = C % 4 == 0 && term_stride % 4 == 0 && al16(slab) && al16(conv_w) && al16(state_in) && al16(state_out) &&
                  al16(x_out) && al16(h_out);
  const int cv = v4 ? C / 4 : C;
  // long runs average fewer tokens twice, short ones give more threads: half of what the SMs hold is enough
  int seg = 16;
  while (seg > 1 && (long long)n_seq * ((T + seg - 1) / seg) * cv < 148ll * 1024) seg >>= 1;
  const int n_seg = (T + seg - 1) / seg;
  const long long work = (long long)n_seq * n_seg * cv;
  const unsigned grid = (unsigned)((work + 127) / 128);
#define DGPT_DC(TT, VV, TP)                                                                                               \
  depth_avg_conv_kernel<TT, VV, TP><<<grid, 128, 0, st>>>(slab, term_stride, terms, coef, conv_w, taps, state_in, state_out, \
                                                          x_out, static_cast<TT*>(h_out), n_seq, T, seg, n_seg, C)
#define DGPT_DCT(TT, VV)                \
  do {                                  \
    if (taps == 1) DGPT_DC(TT, VV, 1);  \
    else if (taps == 2) DGPT_DC(TT, VV, 2); \
    else if (taps == 3) DGPT_DC(TT, VV, 3); \
    else if (taps == 4) DGPT_DC(TT, VV, 4); \
    else if (taps <= 8) DGPT_DC(TT, VV, 8); \
    else DGPT_DC(TT, VV, kMaxTaps);     \
  } while (0)
  if (dtype == DGPT_F32) {
    if (v4) DGPT_DCT(float, 4);
    else DGPT_DCT(float, 1);
  } else {
    if (v4) DGPT_DCT(__nv_bfloat16, 4);
    else DGPT_DCT(__nv_bfloat16, 1);
  }
#undef DGPT_DCT
#undef DGPT_DC
  return launch_status("depth_avg_conv");
}

extern "C" int dgpt_layer_tail(const void* y, const float* norm_w, float eps, const float* x1, float* slab,
                               int64_t term_stride, int32_t terms, const float* coef, const float* conv_w, int32_t taps,
                               float* state, float* x_out, void* h_out, int64_t rows, int32_t C, int32_t dtype, void* stream) {
  DGPT_REQUIRE(y && norm_w && x1 && slab && coef && conv_w && x_out && h_out, "layer_tail: NULL pointer");
  DGPT_REQUIRE(terms >= 2 && rows >= 0 && rows <= 0x7fffffff && C > 0, "layer_tail: bad sizes");
  DGPT_REQUIRE(taps >= 1 && (taps == 1 || state), "layer_tail: the convolution's state is missing");
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, "layer_tail: unknown dtype %d", dtype);
  if (rows == 0) return DGPT_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const long long rows_ = rows;
  const bool v4 = C % 4 == 0 && term_stride % 4 == 0 && al16(y) && al16(norm_w) && al16(x1) && al16(slab) && al16(conv_w) &&
                  al16(state) && al16(x_out) && al16(h_out);
#define DGPT_LT(TT, VV)                                                                                                  \
  DGPT_ROW_DISPATCH(layer_tail_kernel, TT, VV, static_cast<const TT*>(y), norm_w, eps, x1, slab, term_stride, terms, coef, \
                    conv_w, taps, state, x_out, static_cast<TT*>(h_out), C)
  if (dtype == DGPT_F32) {
    if (v4) DGPT_LT(float, 4);
    else DGPT_LT(float, 1);
  } else {
    if (v4) DGPT_LT(__nv_bfloat16, 4);
    else DGPT_LT(__nv_bfloat16, 1);
  }
#undef DGPT_LT
  return launch_status("layer_tail");
}

extern "C" int dgpt_depth_avg_norm(const float* slab, int64_t term_stride, int32_t terms, const float* coef, const float* w,
                                   float eps, const int32_t* row_index, void* out, int64_t n_out, int64_t n, int32_t C,
                                   int32_t dtype, void* stream) {
  DGPT_REQUIRE(slab && coef && w && out, "depth_avg_norm: NULL pointer");
  DGPT_REQUIRE(terms >= 1 && n_out >= 0 && n_out <= 0x7fffffff && n > 0 && C > 0, "depth_avg_norm: bad sizes");
  DGPT_REQUIRE(row_index || n_out <= n, "depth_avg_norm: more rows asked for than there are");
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, "depth_avg_norm: unknown dtype %d", dtype);
  if (n_out == 0) return DGPT_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const long long rows_ = n_out;
  const bool v4 = C % 4 == 0 && term_stride % 4 == 0 && al16(slab) && al16(w) && al16(out);
#define DGPT_DN(TT, VV)                                                                                          \
  DGPT_ROW_DISPATCH(depth_avg_norm_kernel, TT, VV, slab, term_stride, terms, coef, w, eps, row_index, static_cast<TT*>(out), \
                    (long long)n, C)
  if (dtype == DGPT_F32) {
    if (v4) DGPT_DN(float, 4);
    else DGPT_DN(float, 1);
  } else {
    if (v4) DGPT_DN(__nv_bfloat16, 4);
    else DGPT_DN(__nv_bfloat16, 1);
  }
#undef DGPT_DN
  return launch_status("depth_avg_norm");
}

extern "C" int dgpt_xielu(const void* in, void* out, int64_t n, float alpha_p, float alpha_n, int32_t dtype, void* stream) {
  DGPT_REQUIRE(in && out && n >= 0, "xielu: bad arguments");
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, "xielu: unknown dtype %d", dtype);
  if (n == 0) return DGPT_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool v4 = n % 4 == 0 && al16(in) && al16(out);
  const long long work = v4 ? n / 4 : n;
  const unsigned grid = (unsigned)((work + 255) / 256);
#define DGPT_XI(TT, VV) \
  xielu_kernel<TT, VV><<<grid, 256, 0, st>>>(static_cast<const TT*>(in), static_cast<TT*>(out), n, alpha_p, alpha_n)
  if (dtype == DGPT_F32) {
    if (v4) DGPT_XI(float, 4);
    else DGPT_XI(float, 1);
  } else {
    if (v4) DGPT_XI(__nv_bfloat16, 4);
    else DGPT_XI(__nv_bfloat16, 1);
  }
#undef DGPT_XI
  return launch_status("xielu");
}

extern "C" int dgpt_silu_mul(const void* in, void* out, int64_t n_out, int32_t dtype, void* stream) {
  DGPT_REQUIRE(in && out && n_out >= 0, "silu_mul: bad arguments");
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, "silu_mul: unknown dtype %d", dtype);
  if (n_out == 0) return DGPT_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool v4 = n_out % 4 == 0 && al16(in) && al16(out);
  const long long work = v4 ? n_out / 4 : n_out;
  const unsigned grid = (unsigned)((work + 255) / 256);
#define DGPT_SM(TT, VV) silu_mul_kernel<TT, VV><<<grid, 256, 0, st>>>(static_cast<const TT*>(in), static_cast<TT*>(out), n_out)
  if (dtype == DGPT_F32) {
    if (v4) DGPT_SM(float, 4);
    else DGPT_SM(float, 1);
  } else {
    if (v4) DGPT_SM(__nv_bfloat16, 4);
    else DGPT_SM(__nv_bfloat16, 1);
  }
#undef DGPT_SM
  return launch_status("silu_mul");
}
