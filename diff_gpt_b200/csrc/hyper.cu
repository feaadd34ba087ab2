// Row-wise kernels of models whose residual is several fp32 streams (hyper-connections), and the embedding in front of them:
//
//   embed_streams   e = Emb[id] + Big[row(previous id, id)] ; h = rms_norm((sum_s a_s) e) * w      (all streams start as e)
//   streams_step    x'_t = sum_s mix[s, t] x_s + out_t y ;  h = rms_norm(sum_t a_t x'_t) * w       one sublayer to the next
//   streams_final   h = rms_norm(sum_s b_s x_s + c y) * w                                          the rows the head reads
//
// y is a sublayer's output and h the next one's input, in the model dtype; everything else is fp32.  Streams lie
// `stream_stride` elements apart (0: all of them are the same row, as after the embedding).  One CTA per token: each
// stream row is read once and written once, which is what bounds these kernels (HBM); the combined row waits in shared
// memory for its norm.  VEC = 4 channels per thread and step where C is a multiple of 4, 1 otherwise.
#include "rowvec.cuh"

namespace dgpt {

constexpr int kMaxStreams = 16;

// h = u / sqrt(mean(u^2) + eps) * w for the row u in shared memory whose sum of squares is spread over the threads
template <typename T, int VEC>
__device__ __forceinline__ void norm_store(const float* u, float ss, float* scratch, const float* __restrict__ w, float eps,
                                           T* __restrict__ h, int C) {
  const float inv = rsqrtf(block_sum(ss, scratch) / (float)C + eps);
  for (int c = threadIdx.x * VEC; c < C; c += blockDim.x * VEC) {  // a thread reads back what it wrote
    FVec<VEC> v = ldf<VEC>(u + c);
    const FVec<VEC> wv = ldf<VEC>(w + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v.v[e] *= inv * wv.v[e];
    stt<T, VEC>(h + c, v);
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kRowThreads)
embed_streams_kernel(const int* __restrict__ ids, const int* prev_in, int* prev_out, const T* __restrict__ emb, int V,
                     const T* __restrict__ big, long long buckets, long long mul_prev, long long mul_cur,
                     const float* __restrict__ a, int S, const float* __restrict__ w, float eps, float* __restrict__ e_out,
                     T* __restrict__ h, int Tn, int C) {
  extern __shared__ __align__(16) float su[];
  __shared__ float scratch[40];
  const long long row = blockIdx.x;
  const int s = (int)(row / Tn), t = (int)(row - (long long)s * Tn);
  const int id = min(max(ids[row], 0), V - 1);
  int prev = t > 0 ? ids[row - 1] : (prev_in ? prev_in[s] : -1);
  long long b = buckets;  // a sequence's first token has the last row to itself
  if (prev >= 0) b = ((long long)min(prev, V - 1) * mul_prev + (long long)id * mul_cur) % buckets;
  float sum = 0.f;
  for (int i = 0; i < S; ++i) sum += a[i];
  const T* er = emb + (long long)id * C;
  const T* br = big + b * C;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < C; c += blockDim.x * VEC) {
    FVec<VEC> x = ldt<T, VEC>(er + c);
    const FVec<VEC> y = ldt<T, VEC>(br + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) x.v[e] += y.v[e];
    stf<VEC>(e_out + row * C + c, x);
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      x.v[e] *= sum;
      ss += x.v[e] * x.v[e];
    }
    stf<VEC>(su + c, x);
  }
  norm_store<T, VEC>(su, ss, scratch, w, eps, h + row * C, C);  // its barriers also order the read of prev_in
  if (prev_out && t == Tn - 1 && threadIdx.x == 0) prev_out[s] = id;
}

// SM: streams the registers are laid out for (S <= SM).  coef: mix [S, S] (from, to), out [S], in of the next sublayer [S].
template <typename T, int VEC, int SM>
__global__ void __launch_bounds__(kRowThreads)
streams_step_kernel(const float* x, long long x_stride, const T* __restrict__ y, const float* __restrict__ mix,
                    const float* __restrict__ out, const float* __restrict__ a, int S, const float* __restrict__ w, float eps,
                    float* x_new, long long x_new_stride, T* __restrict__ h, int C) {
  extern __shared__ __align__(16) float su[];
  __shared__ float scratch[40], sm[SM * SM + 2 * SM];
  const long long row = blockIdx.x;
  for (int i = threadIdx.x; i < SM * SM + 2 * SM; i += blockDim.x) {  // unused streams get zeros
    float v = 0.f;
    if (i < SM * SM) {
      if (i / SM < S && i % SM < S) v = mix[(i / SM) * S + i % SM];
    } else if (i < SM * SM + SM) {
      if (i - SM * SM < S) v = out[i - SM * SM];
    } else if (i - SM * SM - SM < S) {
      v = a[i - SM * SM - SM];
    }
    sm[i] = v;
  }
  __syncthreads();
  float ss = 0.f;
#pragma unroll 2
  for (int c = threadIdx.x * VEC; c < C; c += blockDim.x * VEC) {
    FVec<VEC> xs[SM];
#pragma unroll
    for (int s = 0; s < SM; ++s) {
      if (s < S) xs[s] = ldf<VEC>(x + s * x_stride + row * C + c);
      else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) xs[s].v[e] = 0.f;
      }
    }
    const FVec<VEC> yv = ldt<T, VEC>(y + row * C + c);
    FVec<VEC> u;
#pragma unroll
    for (int e = 0; e < VEC; ++e) u.v[e] = 0.f;
#pragma unroll
    for (int t = 0; t < SM; ++t) {
      if (t >= S) break;
      FVec<VEC> n;
      const float ot = sm[SM * SM + t], at = sm[SM * SM + SM + t];
#pragma unroll
      for (int e = 0; e < VEC; ++e) n.v[e] = ot * yv.v[e];
#pragma unroll
      for (int s = 0; s < SM; ++s) {
        const float m = sm[s * SM + t];
#pragma unroll
        for (int e = 0; e < VEC; ++e) n.v[e] = fmaf(m, xs[s].v[e], n.v[e]);
      }
      stf<VEC>(x_new + t * x_new_stride + row * C + c, n);
#pragma unroll
      for (int e = 0; e < VEC; ++e) u.v[e] = fmaf(at, n.v[e], u.v[e]);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += u.v[e] * u.v[e];
    if (h) stf<VEC>(su + c, u);
  }
  if (h) norm_store<T, VEC>(su, ss, scratch, w, eps, h + row * C, C);
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kRowThreads)
streams_final_kernel(const float* __restrict__ x, long long x_stride, const T* __restrict__ y, const float* __restrict__ mix,
                     const float* __restrict__ out, int S, const float* __restrict__ w, float eps,
                     const int* __restrict__ row_index, T* __restrict__ h, long long n, int C) {
  extern __shared__ __align__(16) float su[];
  __shared__ float scratch[40];
  const long long row = blockIdx.x;
  long long src = row_index ? (long long)row_index[row] : row;
  src = src < 0 ? 0 : (src >= n ? n - 1 : src);
  float b[kMaxStreams], cy = 0.f;  // the sum of the new streams: stream s enters with sum_t mix[s, t], y with sum_t out[t]
#pragma unroll
  for (int s = 0; s < kMaxStreams; ++s) {
    b[s] = 0.f;
    if (s < S) {
      for (int t = 0; t < S; ++t) b[s] += mix[s * S + t];
      cy += out[s];
    }
  }
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < C; c += blockDim.x * VEC) {
    FVec<VEC> u = ldt<T, VEC>(y + src * C + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) u.v[e] *= cy;
#pragma unroll
    for (int s = 0; s < kMaxStreams; ++s) {
      if (s < S) {
        const FVec<VEC> xv = ldf<VEC>(x + s * x_stride + src * C + c);
#pragma unroll
        for (int e = 0; e < VEC; ++e) u.v[e] = fmaf(b[s], xv.v[e], u.v[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += u.v[e] * u.v[e];
    stf<VEC>(su + c, u);
  }
  norm_store<T, VEC>(su, ss, scratch, w, eps, h + row * C, C);
}

constexpr int kMaxHyperWidth = 12032;  // a row of floats in 47 KB of shared memory

}  // namespace dgpt

using namespace dgpt;

#define DGPT_HC_COMMON(what)                                                                                           \
  DGPT_REQUIRE(C > 0 && C <= kMaxHyperWidth, what ": width must be in [1, %d]", kMaxHyperWidth);                       \
  DGPT_REQUIRE(S >= 1 && S <= kMaxStreams, what ": 1 to %d streams", kMaxStreams);                                     \
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, what ": unknown dtype %d", dtype);                             \
  cudaStream_t st = static_cast<cudaStream_t>(stream);                                                                 \
  using B = __nv_bfloat16;                                                                                             \
  const size_t smem = (size_t)C * 4

extern "C" int dgpt_embed_streams(const int32_t* ids, const int32_t* prev_in, int32_t* prev_out, const void* emb, int32_t V,
                                  const void* big, int64_t buckets, int64_t mul_prev, int64_t mul_cur, const float* a, int32_t S,
                                  const float* w, float eps, float* e_out, void* h, int32_t n_seq, int32_t T, int32_t C,
                                  int32_t dtype, void* stream) {
  DGPT_REQUIRE(ids && emb && big && a && w && e_out && h, "embed_streams: NULL pointer");
  DGPT_REQUIRE(n_seq >= 0 && T >= 0 && V > 0 && buckets > 0 && mul_prev >= 0 && mul_cur >= 0, "embed_streams: bad sizes");
  DGPT_REQUIRE(mul_prev < ((int64_t)1 << 31) && mul_cur < ((int64_t)1 << 31), "embed_streams: multipliers beyond 31 bits");
  DGPT_REQUIRE(prev_in == nullptr || prev_in != prev_out || T <= 1, "embed_streams: the state may be updated in place for T = 1 only");
  DGPT_HC_COMMON("embed_streams");
  const long long n = (long long)n_seq * T;
  if (n == 0) return DGPT_OK;
  const bool v4 = C % 4 == 0 && al16(emb) && al16(big) && al16(w) && al16(e_out) && al16(h);
  const int th = row_threads(v4 ? C / 4 : C);
#define DGPT_ES(TT, VV)                                                                                                     \
  embed_streams_kernel<TT, VV><<<(unsigned)n, th, smem, st>>>(ids, prev_in, prev_out, static_cast<const TT*>(emb), V,      \
                                                              static_cast<const TT*>(big), buckets, mul_prev, mul_cur, a, S, w, \
                                                              eps, e_out, static_cast<TT*>(h), T, C)
  if (dtype == DGPT_F32) {
    if (v4) DGPT_ES(float, 4);
    else DGPT_ES(float, 1);
  } else {
    if (v4) DGPT_ES(B, 4);
    else DGPT_ES(B, 1);
  }
#undef DGPT_ES
  return launch_status("embed_streams");
}

extern "C" int dgpt_streams_step(const float* x, int64_t x_stream_stride, const void* y, const float* mix, const float* out,
                                 const float* a, int32_t S, const float* w, float eps, float* x_new, int64_t x_new_stream_stride,
                                 void* h, int64_t rows, int32_t C, int32_t dtype, void* stream) {
  DGPT_REQUIRE(x && y && mix && out && x_new && (h == nullptr || (a && w)), "streams_step: NULL pointer");
  DGPT_REQUIRE(rows >= 0 && rows <= 0x7fffffff && x_stream_stride >= 0 && (S == 1 || x_new_stream_stride >= rows * C), "streams_step: bad sizes");
  DGPT_REQUIRE(x != x_new || x_stream_stride == x_new_stream_stride, "streams_step: in place needs equal strides");
  DGPT_HC_COMMON("streams_step");
  if (rows == 0) return DGPT_OK;
  if (h == nullptr) a = out;  // not used
  const bool v4 = C % 4 == 0 && x_stream_stride % 4 == 0 && x_new_stream_stride % 4 == 0 && al16(x) && al16(y) && al16(w) &&
                  al16(x_new) && al16(h);
  const int th = row_threads(v4 ? C / 4 : C);
#define DGPT_SS(TT, VV, SS)                                                                                             \
  streams_step_kernel<TT, VV, SS><<<(unsigned)rows, th, smem, st>>>(x, x_stream_stride, static_cast<const TT*>(y), mix, out, a, \
                                                                    S, w, eps, x_new, x_new_stream_stride, static_cast<TT*>(h), C)
#define DGPT_SSV(TT, VV)              \
  do {                                \
    if (S == 1) DGPT_SS(TT, VV, 1);   \
    else if (S == 2) DGPT_SS(TT, VV, 2); \
    else if (S <= 4) DGPT_SS(TT, VV, 4); \
    else if (S <= 8) DGPT_SS(TT, VV, 8); \
    else DGPT_SS(TT, VV, kMaxStreams); \
  } while (0)
  if (dtype == DGPT_F32) {
    if (v4) DGPT_SSV(float, 4);
    else DGPT_SSV(float, 1);
  } else {
    if (v4) DGPT_SSV(B, 4);
    else DGPT_SSV(B, 1);
  }
#undef DGPT_SSV
#undef DGPT_SS
  return launch_status("streams_step");
}

extern "C" int dgpt_streams_final(const float* x, int64_t x_stream_stride, const void* y, const float* mix, const float* out,
                                  int32_t S, const float* w, float eps, const int32_t* row_index, void* h, int64_t n_out, int64_t n,
                                  int32_t C, int32_t dtype, void* stream) {
  DGPT_REQUIRE(x && y && mix && out && w && h, "streams_final: NULL pointer");
  DGPT_REQUIRE(n_out >= 0 && n_out <= 0x7fffffff && n > 0 && x_stream_stride >= 0, "streams_final: bad sizes");
  DGPT_REQUIRE(row_index || n_out <= n, "streams_final: more rows asked for than there are");
  DGPT_HC_COMMON("streams_final");
  if (n_out == 0) return DGPT_OK;
  const bool v4 = C % 4 == 0 && x_stream_stride % 4 == 0 && al16(x) && al16(y) && al16(w) && al16(h);
  const int th = row_threads(v4 ? C / 4 : C);
#define DGPT_SF(TT, VV)                                                                                                  \
  streams_final_kernel<TT, VV><<<(unsigned)n_out, th, smem, st>>>(x, x_stream_stride, static_cast<const TT*>(y), mix, out, S, w, \
                                                                  eps, row_index, static_cast<TT*>(h), (long long)n, C)
  if (dtype == DGPT_F32) {
    if (v4) DGPT_SF(float, 4);
    else DGPT_SF(float, 1);
  } else {
    if (v4) DGPT_SF(B, 4);
    else DGPT_SF(B, 1);
  }
#undef DGPT_SF
  return launch_status("streams_final");
}
