// RoPE + QK RMSNorm + KV-cache append, one warp per (token, head).
//
// Each lane owns rotation pairs  p = lane, lane + 32, ...  (< D/2), i.e. elements
// (2p, 2p+1): a 4-byte (bf16) or 8-byte (fp32) access per lane, consecutive across
// the warp.  q is written to a dense [token, H*D] buffer, k and v go straight into
// their cache page, so the projection output is read once and the cache written once.
#include "common.cuh"

namespace dgpt {

template <typename T>
struct Pair;
template <>
struct Pair<float> {
  static __device__ __forceinline__ float2 ld(const float* p) { return *reinterpret_cast<const float2*>(p); }
  static __device__ __forceinline__ void st(float* p, float a, float b) {
    *reinterpret_cast<float2*>(p) = make_float2(a, b);
  }
};
template <>
struct Pair<__nv_bfloat16> {
  static __device__ __forceinline__ float2 ld(const __nv_bfloat16* p) {
    return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
  }
  static __device__ __forceinline__ void st(__nv_bfloat16* p, float a, float b) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
  }
};

constexpr int kMaxPairsPerLane = 4;  // head_dim <= 256

template <typename T>
__global__ void rope_qknorm_kvappend_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v,
                                            long long in_stride, T* __restrict__ q_out, long long q_out_stride,
                                            const T* __restrict__ cs, int table_len, KvView kv,
                                            const int* __restrict__ seq_pos0, const int* __restrict__ seq_slot0,
                                            const int* __restrict__ step_ptr, int n_seq, int T_len, int H, int D,
                                            int* __restrict__ status) {
  const long long wid = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const long long total = (long long)n_seq * T_len * H;
  if (wid >= total) return;
  const int lane = threadIdx.x & 31;
  const int h = (int)(wid % H);
  const long long tok = wid / H;
  const int s = (int)(tok / T_len), t = (int)(tok - (long long)s * T_len);
  const int step = step_ptr ? *step_ptr : 0;
  const int pos = seq_pos0[s] + step + t;
  const int slot = seq_slot0[s] + step + t;
  const int cap = kv.page_table ? kv.max_pages * kv.page_tokens : kv.page_tokens;
  if (pos < 0 || pos >= table_len || slot < 0 || slot >= cap) {
    if (lane == 0) atomicExch(status, 1);
    return;
  }
  const int half = D >> 1;
  const T* qs = q + tok * in_stride + (long long)h * D;
  const T* ks = k + tok * in_stride + (long long)h * D;
  const T* vs = v + tok * in_stride + (long long)h * D;
  const T* csr = cs + (long long)pos * D;  // (D/2, 2) per position

  float qa[kMaxPairsPerLane], qb[kMaxPairsPerLane], ka[kMaxPairsPerLane], kb[kMaxPairsPerLane];
  float qss = 0.f, kss = 0.f;
#pragma unroll
  for (int i = 0; i < kMaxPairsPerLane; ++i) {
    const int p = lane + 32 * i;
    qa[i] = qb[i] = ka[i] = kb[i] = 0.f;
    if (p < half) {
      const float2 c = Pair<T>::ld(csr + 2 * p);  // (cos, sin), upcast from the storage type
      const float2 x = Pair<T>::ld(qs + 2 * p);
      const float2 y = Pair<T>::ld(ks + 2 * p);
      qa[i] = Io<T>::round(x.x * c.x - x.y * c.y);
      qb[i] = Io<T>::round(x.x * c.y + x.y * c.x);
      ka[i] = Io<T>::round(y.x * c.x - y.y * c.y);
      kb[i] = Io<T>::round(y.x * c.y + y.y * c.x);
      qss += qa[i] * qa[i] + qb[i] * qb[i];
      kss += ka[i] * ka[i] + kb[i] * kb[i];
    }
  }
  qss = warp_sum(qss);
  kss = warp_sum(kss);
  const float qinv = rsqrtf(qss / (float)D + kRmsEps);
  const float kinv = rsqrtf(kss / (float)D + kRmsEps);

  const long long off = kv_offset(kv, s, h, slot, D);
  T* kd = static_cast<T*>(kv.k) + off;
  T* vd = static_cast<T*>(kv.v) + off;
  T* qd = q_out + tok * q_out_stride + (long long)h * D;
#pragma unroll
  for (int i = 0; i < kMaxPairsPerLane; ++i) {
    const int p = lane + 32 * i;
    if (p < half) {
      Pair<T>::st(qd + 2 * p, qa[i] * qinv, qb[i] * qinv);
      Pair<T>::st(kd + 2 * p, ka[i] * kinv, kb[i] * kinv);
      const float2 vv = Pair<T>::ld(vs + 2 * p);
      Pair<T>::st(vd + 2 * p, vv.x, vv.y);
    }
  }
}

// Vector variant: LPH = D / VEC lanes own one (token, head), each lane one 16-byte vector (VEC / 2
// rotation pairs) of q, k, v and of the (cos, sin) row, so a warp covers 32 / LPH heads and every
// access is 16 bytes wide.  Same rounding points as the scalar kernel.
template <typename T, int D>
__global__ void rope_qknorm_kvappend_vec_kernel(const T* __restrict__ q, const T* __restrict__ k,
                                                const T* __restrict__ v, long long in_stride, T* __restrict__ q_out,
                                                long long q_out_stride, const T* __restrict__ cs, int table_len,
                                                KvView kv, const int* __restrict__ seq_pos0,
                                                const int* __restrict__ seq_slot0, const int* __restrict__ step_ptr,
                                                int n_seq, int T_len, int H, int* __restrict__ status) {
  constexpr int VEC = Io<T>::kVec16;
  constexpr int LPH = D / VEC;
  static_assert(LPH >= 1 && LPH <= 32 && (LPH & (LPH - 1)) == 0, "unsupported head_dim");
  dep_wait();
  const long long unit = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / LPH;  // (token, head)
  const int e = threadIdx.x % LPH;
  const long long total = (long long)n_seq * T_len * H;
  const bool live = unit < total;
  const long long u = live ? unit : total - 1;  // idle lanes shadow the last unit so that shuffles stay full
  const int h = (int)(u % H);
  const long long tok = u / H;
  const int s = (int)(tok / T_len), t = (int)(tok - (long long)s * T_len);
  const int step = step_ptr ? *step_ptr : 0;
  const int pos = seq_pos0[s] + step + t;
  const int slot = seq_slot0[s] + step + t;
  const int cap = kv.page_table ? kv.max_pages * kv.page_tokens : kv.page_tokens;
  const bool in_range = pos >= 0 && pos < table_len && slot >= 0 && slot < cap;
  if (live && !in_range && e == 0) atomicExch(status, 1);
  const int pos_c = in_range ? pos : 0;
  const long long src = tok * in_stride + (long long)h * D + e * VEC;
  float qf[VEC], kf[VEC], cf[VEC];
  ld16<T>(q + src, qf);
  ld16<T>(k + src, kf);
  ld16<T>(cs + (long long)pos_c * D + e * VEC, cf);  // (cos, sin) pairs of this lane's rotation pairs
  const uint4 vraw = *reinterpret_cast<const uint4*>(v + src);
  float qss = 0.f, kss = 0.f;
#pragma unroll
  for (int i = 0; i < VEC; i += 2) {
    const float c = cf[i], sn = cf[i + 1];
    const float qa = Io<T>::round(qf[i] * c - qf[i + 1] * sn), qb = Io<T>::round(qf[i] * sn + qf[i + 1] * c);
    const float ka = Io<T>::round(kf[i] * c - kf[i + 1] * sn), kb = Io<T>::round(kf[i] * sn + kf[i + 1] * c);
    qf[i] = qa; qf[i + 1] = qb; kf[i] = ka; kf[i + 1] = kb;
    qss += qa * qa + qb * qb;
    kss += ka * ka + kb * kb;
  }
#pragma unroll
  for (int o = LPH >> 1; o > 0; o >>= 1) {
    qss += __shfl_xor_sync(0xffffffffu, qss, o);
    kss += __shfl_xor_sync(0xffffffffu, kss, o);
  }
  if (!live || !in_range) return;
  const float qinv = rsqrtf(qss / (float)D + kRmsEps);
  const float kinv = rsqrtf(kss / (float)D + kRmsEps);
  const long long off = kv_offset(kv, s, h, slot, D) + e * VEC;
  st16<T>(q_out + tok * q_out_stride + (long long)h * D + e * VEC, qf, qinv);
  st16<T>(static_cast<T*>(kv.k) + off, kf, kinv);
  *reinterpret_cast<uint4*>(static_cast<T*>(kv.v) + off) = vraw;
}

template <typename T, int D>
static int rope_vec_launch(const void* q, const void* k, const void* v, long long in_stride, void* q_out,
                           long long q_out_stride, const void* cs, int table_len, const KvView& view,
                           const int* pos0, const int* slot0, const int* step_ptr, int n_seq, int T_len, int H,
                           int* status, cudaStream_t st) {
  constexpr int LPH = D / Io<T>::kVec16;
  const long long threads = (long long)n_seq * T_len * H * LPH;
  const unsigned grid = (unsigned)((threads + 255) / 256);
  launch_dep(rope_qknorm_kvappend_vec_kernel<T, D>, dim3(grid), dim3(256), 0, st, static_cast<const T*>(q),
             static_cast<const T*>(k), static_cast<const T*>(v), in_stride, static_cast<T*>(q_out), q_out_stride,
             static_cast<const T*>(cs), table_len, view, pos0, slot0, step_ptr, n_seq, T_len, H, status);
  return launch_status("rope_qknorm_kvappend");
}

// ---- norm over whole projections, rotation of the leading dimensions, append to a cache of rows ------------------
// CTA per token.  q and k are normalised over all their heads at once, then the first `rot` dimensions of each head are
// rotated in interleaved pairs; the cache row is [keys of G heads | values of G heads].  A thread takes four dimensions of a
// head at a time (heads are a multiple of 8 wide), which hold two whole pairs.
constexpr int kRowsThreads = 256;
template <typename T>
__device__ __forceinline__ void ld4(const T* p, float* v);
template <>
__device__ __forceinline__ void ld4<float>(const float* p, float* v) {
  const float4 t = *reinterpret_cast<const float4*>(p);
  v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
}
template <>
__device__ __forceinline__ void ld4<__nv_bfloat16>(const __nv_bfloat16* p, float* v) {
  const uint2 t = *reinterpret_cast<const uint2*>(p);
  v[0] = __uint_as_float(t.x << 16); v[1] = __uint_as_float(t.x & 0xffff0000u);
  v[2] = __uint_as_float(t.y << 16); v[3] = __uint_as_float(t.y & 0xffff0000u);
}
template <typename T>
__device__ __forceinline__ void st4(T* p, const float* v) {
  Pair<T>::st(p, v[0], v[1]);
  Pair<T>::st(p + 2, v[2], v[3]);
}

// where the cache row of slot `slot` of sequence s lies, or NULL
template <typename T>
__device__ __forceinline__ T* cache_row(const KvView& kv, int s, int slot, int row_w) {
  const int cap = kv.page_table ? kv.max_pages * kv.page_tokens : kv.page_tokens;
  if (slot < 0 || slot >= cap) return nullptr;
  const int lp = slot / kv.page_tokens;
  long long pg = s;
  if (kv.page_table) pg = kv.page_table[(long long)s * kv.max_pages + lp];
  if (pg < 0 || (kv.n_pages > 0 && pg >= kv.n_pages)) return nullptr;
  return static_cast<T*>(kv.k) + pg * kv.page_stride + (long long)(slot - lp * kv.page_tokens) * row_w;
}

struct ProjArgs {
  long long in_rs, q_rs;
  const float *qw, *kw;
  float q_count, k_count, eps;
  const float2* table;
  int table_len, rot, row_w;
  const int *pos0, *slot0, *step_ptr;
  int Tn, HD, GD, GE, D;
  int* status;
};

// One warp per token, q and k of the token in registers as they were loaded (NV 16-byte pieces per lane).
template <typename T, int NV>
__global__ void __launch_bounds__(256)
proj_norm_rope_append_warp_kernel(const T* __restrict__ in, T* __restrict__ q_out, const KvView kv, const ProjArgs a, long long n_tok) {
  constexpr int VEC = Io<T>::kVec16;
  const long long tok = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (tok >= n_tok) return;
  const int lane = threadIdx.x & 31;
  const int s = (int)(tok / a.Tn), t = (int)(tok - (long long)s * a.Tn);
  const T* row = in + tok * a.in_rs;
  const int n = a.HD + a.GD;
  uint4 raw[NV];
  float qs = 0.f, ks = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (lane + 32 * i) * VEC;
    raw[i] = make_uint4(0u, 0u, 0u, 0u);
    if (c < n) raw[i] = __ldg(reinterpret_cast<const uint4*>(row + c));
  }
  const int step = a.step_ptr ? *a.step_ptr : 0;
  const int pos = a.pos0[s] + step + t;
  T* dst = cache_row<T>(kv, s, a.slot0[s] + step + t, a.row_w);
  const bool ok = pos >= 0 && pos < a.table_len;
  if ((dst == nullptr || !ok) && lane == 0 && a.status) *a.status = 1;
  const float2* cs = a.table + (long long)(ok ? pos : 0) * (a.rot >> 1);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (lane + 32 * i) * VEC;
    float v[VEC], ss = 0.f;
    unpack16<T>(raw[i], v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += v[e] * v[e];
    if (c < a.HD) qs += ss;
    else ks += ss;
  }
  const float qi = rsqrtf(warp_sum(qs) / a.q_count + a.eps), ki = rsqrtf(warp_sum(ks) / a.k_count + a.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (lane + 32 * i) * VEC;
    if (c >= n) continue;
    const bool is_q = c < a.HD;
    const int x = is_q ? c : c - a.HD, d = x % a.D;
    const float inv = is_q ? qi : ki;
    const float* w = (is_q ? a.qw : a.kw) + x;
    float v[VEC];
    unpack16<T>(raw[i], v);
#pragma unroll
    for (int e = 0; e < VEC; e += 4) {
      const float4 f = __ldg(reinterpret_cast<const float4*>(w + e));
      v[e] *= inv * f.x; v[e + 1] *= inv * f.y; v[e + 2] *= inv * f.z; v[e + 3] *= inv * f.w;
    }
#pragma unroll
    for (int e = 0; e < VEC; e += 2) {
      if (d + e < a.rot) {
        const float2 f = __ldg(cs + ((d + e) >> 1));
        const float p = v[e], q = v[e + 1];
        v[e] = p * f.x - q * f.y;
        v[e + 1] = q * f.x + p * f.y;
      }
    }
    if (is_q) st16<T>(q_out + tok * a.q_rs + x, v, 1.f);
    else if (dst) st16<T>(dst + x, v, 1.f);
  }
  if (dst)
    for (int c = lane * VEC; c < a.GE; c += 32 * VEC)
      *reinterpret_cast<uint4*>(dst + a.GD + c) = __ldg(reinterpret_cast<const uint4*>(row + n + c));
}

// CTA per token, rows of any length.
template <typename T>
__global__ void __launch_bounds__(kRowsThreads)
proj_norm_rope_append_kernel(const T* __restrict__ in, T* __restrict__ q_out, const KvView kv, const ProjArgs a) {
  __shared__ float scratch[40], scratch2[40];
  const long long tok = blockIdx.x;
  const int s = (int)(tok / a.Tn), t = (int)(tok - (long long)s * a.Tn), tid = threadIdx.x;
  const int step = a.step_ptr ? *a.step_ptr : 0;
  const int pos = a.pos0[s] + step + t;
  T* dst = cache_row<T>(kv, s, a.slot0[s] + step + t, a.row_w);
  const bool ok = pos >= 0 && pos < a.table_len;
  if ((dst == nullptr || !ok) && tid == 0 && a.status) *a.status = 1;
  const float2* cs = a.table + (long long)(ok ? pos : 0) * (a.rot >> 1);
  const T* row = in + tok * a.in_rs;
  const int n = a.HD + a.GD;
  float qs = 0.f, ks = 0.f;
  for (int c = tid * 4; c < n; c += kRowsThreads * 4) {
    float v[4];
    ld4<T>(row + c, v);
    const float ss = v[0] * v[0] + v[1] * v[1] + v[2] * v[2] + v[3] * v[3];
    if (c < a.HD) qs += ss;
    else ks += ss;
  }
  qs = block_sum(qs, scratch);
  ks = block_sum(ks, scratch2);
  const float qi = rsqrtf(qs / a.q_count + a.eps), ki = rsqrtf(ks / a.k_count + a.eps);
  for (int c = tid * 4; c < n; c += kRowsThreads * 4) {
    const bool is_q = c < a.HD;
    const int x = is_q ? c : c - a.HD, d = x % a.D;
    float v[4];
    ld4<T>(row + c, v);  // in L1 from the first pass
    const float4 w = *reinterpret_cast<const float4*>((is_q ? a.qw : a.kw) + x);
    const float inv = is_q ? qi : ki;
    v[0] *= inv * w.x; v[1] *= inv * w.y; v[2] *= inv * w.z; v[3] *= inv * w.w;
#pragma unroll
    for (int p = 0; p < 2; ++p) {
      if (d + 2 * p < a.rot) {
        const float2 f = cs[(d >> 1) + p];
        const float x0 = v[2 * p], x1 = v[2 * p + 1];
        v[2 * p] = x0 * f.x - x1 * f.y;
        v[2 * p + 1] = x1 * f.x + x0 * f.y;
      }
    }
    if (is_q) st4<T>(q_out + tok * a.q_rs + x, v);
    else if (dst) st4<T>(dst + x, v);
  }
  if (dst) {
    for (int c = tid * 4; c < a.GE; c += kRowsThreads * 4) {
      float v[4];
      ld4<T>(row + n + c, v);
      st4<T>(dst + a.GD + c, v);
    }
  }
}

template <typename T>
static int proj_launch(const void* in, void* q_out, const KvView& view, const ProjArgs& a, long long n_tok, cudaStream_t st) {
  const T* x = static_cast<const T*>(in);
  T* q = static_cast<T*>(q_out);
  const int nv = (a.HD + a.GD + 32 * Io<T>::kVec16 - 1) / (32 * Io<T>::kVec16);
  const unsigned grid = (unsigned)((n_tok + 7) / 8);
  if (n_tok < 148 * 8 || nv > 16) proj_norm_rope_append_kernel<T><<<(unsigned)n_tok, kRowsThreads, 0, st>>>(x, q, view, a);  // few tokens: a CTA each
  else if (nv <= 2) proj_norm_rope_append_warp_kernel<T, 2><<<grid, 256, 0, st>>>(x, q, view, a, n_tok);
  else if (nv <= 4) proj_norm_rope_append_warp_kernel<T, 4><<<grid, 256, 0, st>>>(x, q, view, a, n_tok);
  else if (nv <= 6) proj_norm_rope_append_warp_kernel<T, 6><<<grid, 256, 0, st>>>(x, q, view, a, n_tok);
  else if (nv <= 8) proj_norm_rope_append_warp_kernel<T, 8><<<grid, 256, 0, st>>>(x, q, view, a, n_tok);
  else if (nv <= 12) proj_norm_rope_append_warp_kernel<T, 12><<<grid, 256, 0, st>>>(x, q, view, a, n_tok);
  else proj_norm_rope_append_warp_kernel<T, 16><<<grid, 256, 0, st>>>(x, q, view, a, n_tok);
  return launch_status("proj_norm_rope_append");
}

}  // namespace dgpt

using namespace dgpt;

extern "C" int dgpt_rope_qknorm_kvappend(const void* q, const void* k, const void* v, int64_t in_row_stride,
                                         void* q_out, int64_t q_out_row_stride, const void* cs_table,
                                         int32_t table_len, const dgpt_kv_layout* kv, const int32_t* seq_pos0,
                                         const int32_t* seq_slot0, const int32_t* step_ptr, int32_t n_seq,
                                         int32_t T, int32_t H, int32_t D, int32_t dtype, int32_t* status,
                                         void* stream) {
  DGPT_REQUIRE(q && k && v && q_out && cs_table && seq_pos0 && seq_slot0 && status, "rope_qknorm_kvappend: NULL pointer");
  DGPT_REQUIRE(n_seq >= 0 && T >= 0 && H > 0, "rope_qknorm_kvappend: bad sizes");
  DGPT_REQUIRE(D > 0 && D % 2 == 0 && D <= 64 * kMaxPairsPerLane, "rope_qknorm_kvappend: head_dim must be even and <= 256");
  DGPT_REQUIRE(in_row_stride % 2 == 0 && q_out_row_stride % 2 == 0, "rope_qknorm_kvappend: row strides must be even");
  if (int e = validate_kv(kv, D)) return e;
  const long long total = (long long)n_seq * T * H;
  if (total == 0) return DGPT_OK;
  const int warps = 8;
  const unsigned grid = (unsigned)((total + warps - 1) / warps);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const KvView view = make_view(kv);
  {
    auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const int vec = dtype == DGPT_BF16 ? 8 : 4;
    const bool aligned = al(q) && al(k) && al(v) && al(q_out) && al(cs_table) && in_row_stride % vec == 0 &&
                         q_out_row_stride % vec == 0 && D % vec == 0;
#define DGPT_ROPE(TT, DD)                                                                                         \
  return rope_vec_launch<TT, DD>(q, k, v, in_row_stride, q_out, q_out_row_stride, cs_table, table_len, view,      \
                                 seq_pos0, seq_slot0, step_ptr, n_seq, T, H, status, st)
    if (aligned && dtype == DGPT_BF16) {
      switch (D) {
        case 8: DGPT_ROPE(__nv_bfloat16, 8);
        case 16: DGPT_ROPE(__nv_bfloat16, 16);
        case 32: DGPT_ROPE(__nv_bfloat16, 32);
        case 64: DGPT_ROPE(__nv_bfloat16, 64);
        case 128: DGPT_ROPE(__nv_bfloat16, 128);
      }
    } else if (aligned && dtype == DGPT_F32) {
      switch (D) {
        case 8: DGPT_ROPE(float, 8);
        case 16: DGPT_ROPE(float, 16);
        case 32: DGPT_ROPE(float, 32);
        case 64: DGPT_ROPE(float, 64);
        case 128: DGPT_ROPE(float, 128);
      }
    }
#undef DGPT_ROPE
  }
  if (dtype == DGPT_F32) {
    rope_qknorm_kvappend_kernel<float><<<grid, warps * 32, 0, st>>>(
        static_cast<const float*>(q), static_cast<const float*>(k), static_cast<const float*>(v), in_row_stride,
        static_cast<float*>(q_out), q_out_row_stride, static_cast<const float*>(cs_table), table_len, view, seq_pos0,
        seq_slot0, step_ptr, n_seq, T, H, D, status);
  } else if (dtype == DGPT_BF16) {
    using B = __nv_bfloat16;
    rope_qknorm_kvappend_kernel<B><<<grid, warps * 32, 0, st>>>(
        static_cast<const B*>(q), static_cast<const B*>(k), static_cast<const B*>(v), in_row_stride,
        static_cast<B*>(q_out), q_out_row_stride, static_cast<const B*>(cs_table), table_len, view, seq_pos0, seq_slot0,
        step_ptr, n_seq, T, H, D, status);
  } else {
    set_error("rope_qknorm_kvappend: unknown dtype %d", dtype);
    return DGPT_E_UNSUPPORTED;
  }
  return launch_status("rope_qknorm_kvappend");
}

extern "C" int dgpt_proj_norm_rope_append(const void* in, int64_t in_row_stride, const float* q_weight, const float* k_weight,
                                          int32_t q_count, int32_t k_count, float eps, const float* table, int32_t table_len,
                                          int32_t rot_dims, void* q_out, int64_t q_out_row_stride, const dgpt_kv_layout* kv,
                                          int32_t row_width, const int32_t* seq_pos0, const int32_t* seq_slot0,
                                          const int32_t* step_ptr, int32_t n_seq, int32_t T, int32_t H, int32_t G, int32_t D,
                                          int32_t Dv, int32_t dtype, int32_t* status, void* stream) {
  DGPT_REQUIRE(in && q_weight && k_weight && table && q_out && seq_pos0 && seq_slot0, "proj_norm_rope_append: NULL pointer");
  DGPT_REQUIRE(n_seq >= 0 && T >= 0 && H > 0 && G > 0 && D > 0 && D % 8 == 0 && Dv > 0 && Dv % 8 == 0 && q_count > 0 && k_count > 0,
               "proj_norm_rope_append: bad sizes (heads must be a multiple of 8 wide)");
  DGPT_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= D && table_len > 0, "proj_norm_rope_append: bad rotation");
  DGPT_REQUIRE(in_row_stride % 8 == 0 && q_out_row_stride % 8 == 0 && row_width % 8 == 0 && row_width >= G * (D + Dv),
               "proj_norm_rope_append: row strides must be multiples of 8");
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  DGPT_REQUIRE(al(in) && al(q_weight) && al(k_weight) && al(q_out), "proj_norm_rope_append: pointers must be 16-byte aligned");
  if (int e = validate_kv(kv, D)) return e;
  const long long n = (long long)n_seq * T;
  if (n == 0) return DGPT_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ProjArgs a;
  a.in_rs = in_row_stride; a.q_rs = q_out_row_stride;
  a.qw = q_weight; a.kw = k_weight;
  a.q_count = (float)q_count; a.k_count = (float)k_count; a.eps = eps;
  a.table = reinterpret_cast<const float2*>(table); a.table_len = table_len; a.rot = rot_dims; a.row_w = row_width;
  a.pos0 = seq_pos0; a.slot0 = seq_slot0; a.step_ptr = step_ptr;
  a.Tn = T; a.HD = H * D; a.GD = G * D; a.GE = G * Dv; a.D = D;
  a.status = status;
  if (dtype == DGPT_F32) return proj_launch<float>(in, q_out, make_view(kv), a, n, st);
  if (dtype == DGPT_BF16) return proj_launch<__nv_bfloat16>(in, q_out, make_view(kv), a, n, st);
  set_error("proj_norm_rope_append: unknown dtype %d", dtype);
  return DGPT_E_UNSUPPORTED;
}
