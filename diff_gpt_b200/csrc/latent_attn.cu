// Attention over cached rows, few queries per sequence (decoding, short portions), with a sliding window and a number of
// first tokens that stay visible.  Two kinds of row (see latent_attn.cuh):
//   latents       one vector of r numbers per token, shared by all heads, with the key and value expansions absorbed into
//                 the query and the output: q~_h = W_uk,h^T q_h and o_h = W_uv,h (sum_j p_j c_j), so scores and sums are
//                 formed on the latents themselves
//   keys, values  of G groups of heads (grouped-query attention)
// Either way a cached row is read once for all heads that share it.
//
//   latent_append_kernel   c = rms_norm(x) * w, rounded once, into the paged cache (and a flat copy where asked for)
//   latent_tc_kernel       latent_tc.cu: bf16 on tcgen05, the form that serves
//   latent_attn_kernel     any r, storage type and page size (fp32 models): scores and sums in fp32 on the CUDA cores
//   latent_combine_kernel  merges key splits
#include "latent_attn.cuh"

namespace dgpt {

constexpr int kLatThreads = 256;

// this split's part [begin, end) of the keys a row sees, counted along [0, ks) and then [lo, n)
struct LatentSpan {
  LatentKeys k;
  int begin, end;
};
__device__ __forceinline__ LatentSpan latent_span(const LatentArgs& a, int row, int split) {
  LatentSpan sp;
  sp.k = latent_keys(a, row);
  const int seen = sp.k.ks + sp.k.n - sp.k.lo;
  const int chunk = (seen + a.n_splits - 1) / a.n_splits;
  sp.begin = min(seen, split * chunk);
  sp.end = min(seen, sp.begin + chunk);
  return sp;
}
// Element offset of the cache row of seen key j, or -1 when its table entry lies outside the pool (such a row counts as zeros).
__device__ __forceinline__ long long latent_offset(const LatentArgs& a, const LatentKeys& k, int j) {
  const int i = j < k.ks ? j : k.lo + (j - k.ks);
  const int slot = i < k.n0 ? i : k.s1 + (i - k.n0);
  const int lp = slot / a.kv.page_tokens;
  const int in = slot - lp * a.kv.page_tokens;
  long long pg = k.seq;
  if (a.kv.page_table) {
    pg = a.kv.page_table[(long long)k.seq * a.kv.max_pages + lp];
    if (a.kv.n_pages > 0 && (pg < 0 || pg >= a.kv.n_pages)) return -1;
  }
  return pg * a.kv.page_stride + (long long)in * a.row_w;
}

// ---- append: one warp per token ---------------------------------------------------------------
// NV > 0: 16-byte accesses, NV of them per lane, the row stays in registers between the two passes; NV = 0: any sizes.
template <typename T, int NV>
__global__ void latent_append_kernel(const T* __restrict__ in, long long in_rs, const float* __restrict__ w, float eps, int r_norm,
                                     KvView kv, const int* __restrict__ slot0, const int* __restrict__ step_ptr, int n_seq, int Tn,
                                     int r, T* __restrict__ flat, int* status) {
  const long long tok = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (tok >= (long long)n_seq * Tn) return;
  const int lane = threadIdx.x & 31;
  const int s = (int)(tok / Tn), t = (int)(tok - (long long)s * Tn);
  const T* x = in + tok * in_rs;
  constexpr int VEC = Io<T>::kVec16, E = NV > 0 ? NV * VEC : 1;
  float val[E];
  float ss = 0.f;
  if constexpr (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (lane + 32 * i) * VEC;
#pragma unroll
      for (int e = 0; e < VEC; ++e) val[i * VEC + e] = 0.f;
      if (c < r_norm) ld16<T>(x + c, val + i * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += val[i * VEC + e] * val[i * VEC + e];
    }
  } else {
    for (int c = lane; c < r_norm; c += 32) {
      const float v = Io<T>::ld(x + c);
      ss += v * v;
    }
  }
  const float inv = rsqrtf(warp_sum(ss) / (float)r_norm + eps);
  const int slot = slot0[s] + (step_ptr ? *step_ptr : 0) + t;
  const int cap = kv.page_table ? kv.max_pages * kv.page_tokens : kv.page_tokens;
  T* dst = nullptr;
  if (slot >= 0 && slot < cap) {
    const int lp = slot / kv.page_tokens;
    long long pg = s;
    if (kv.page_table) pg = kv.page_table[(long long)s * kv.max_pages + lp];
    if (pg >= 0 && (kv.n_pages <= 0 || pg < kv.n_pages))
      dst = static_cast<T*>(kv.k) + pg * kv.page_stride + (long long)(slot - lp * kv.page_tokens) * r;
  }
  if (dst == nullptr && lane == 0 && status) *status = 1;
  if constexpr (NV > 0) {  // r == r_norm
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (lane + 32 * i) * VEC;
      if (c >= r) continue;
#pragma unroll
      for (int e = 0; e < VEC; e += 4) {
        const float4 wv = *reinterpret_cast<const float4*>(w + c + e);
        val[i * VEC + e] *= wv.x;
        val[i * VEC + e + 1] *= wv.y;
        val[i * VEC + e + 2] *= wv.z;
        val[i * VEC + e + 3] *= wv.w;
      }
      if (dst) st16<T>(dst + c, val + i * VEC, inv);
      if (flat) st16<T>(flat + tok * r + c, val + i * VEC, inv);
    }
    return;
  }
  for (int c = lane; c < r; c += 32) {
    const float v = c < r_norm ? Io<T>::ld(x + c) * inv * w[c] : 0.f;
    if (dst) Io<T>::st(dst + c, v);
    if (flat) Io<T>::st(flat + tok * r + c, v);
  }
}

// ---- any sizes, any storage type, CUDA cores ------------------------------------------------------
// Shared memory: q and o of `hg` heads of one group in fp32, a tile of `tt` keys (row stride dk + 1) and of their values
// (dv + 1; the same tile where the values are the keys), scores.
template <typename T>
__global__ void __launch_bounds__(kLatThreads) latent_attn_kernel(const LatentArgs a, int hg, int tt) {
  extern __shared__ __align__(16) uint8_t lat_raw[];
  const int dk = a.dk, dv = a.dv, ldk = dk + 1, ldv = dv + 1;
  const bool same = a.v_col == 0;
  float* sq = reinterpret_cast<float*>(lat_raw);  // [hg][dk]
  float* so = sq + hg * dk;                       // [hg][dv]
  float* sk = so + hg * dv;                       // [tt][dk + 1]
  float* sv = same ? sk : sk + tt * ldk;          // [tt][dv + 1]
  float* sp_ = sv + tt * ldv;                     // [hg][tt]
  float* sm = sp_ + hg * tt;                      // [hg] running maximum, [hg] sum, [hg] rescale
  const int tid = threadIdx.x;
  const int row = blockIdx.x, split = blockIdx.y;
  const int per = a.H / a.G, n_hg = (per + hg - 1) / hg;
  const int g = blockIdx.z / n_hg, hi = (blockIdx.z - g * n_hg) * hg;
  const int h0 = g * per + hi, nh = min(hg, per - hi);
  const LatentSpan sp = latent_span(a, row, split);
  const T* q = static_cast<const T*>(a.q) + (long long)row * a.q_rs + (long long)h0 * dk;
  for (int i = tid; i < nh * dk; i += kLatThreads) sq[i] = Io<T>::ld(q + i) * a.scale_log2;
  for (int i = tid; i < nh * dv; i += kLatThreads) so[i] = 0.f;
  if (tid < nh) {
    sm[tid] = -INFINITY;
    sm[hg + tid] = 0.f;
  }
  const T* pool = static_cast<const T*>(a.kv.k);
  for (int i0 = sp.begin; i0 < sp.end; i0 += tt) {
    const int cnt = min(tt, sp.end - i0);
    __syncthreads();
    for (int t = tid >> 5; t < cnt; t += kLatThreads / 32) {
      const long long off = latent_offset(a, sp.k, i0 + t);
      const T* src = pool + off + g * dk;
      for (int c = tid & 31; c < dk; c += 32) sk[t * ldk + c] = off < 0 ? 0.f : Io<T>::ld(src + c);
      if (!same) {
        src = pool + off + a.v_col + g * dv;
        for (int c = tid & 31; c < dv; c += 32) sv[t * ldv + c] = off < 0 ? 0.f : Io<T>::ld(src + c);
      }
    }
    __syncthreads();
    for (int i = tid; i < nh * cnt; i += kLatThreads) {
      const int h = i / cnt, t = i - h * cnt;
      const float* qh = sq + h * dk;
      const float* ct = sk + t * ldk;
      float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
      int c = 0;
      for (; c + 4 <= dk; c += 4) {
        d0 += qh[c] * ct[c];
        d1 += qh[c + 1] * ct[c + 1];
        d2 += qh[c + 2] * ct[c + 2];
        d3 += qh[c + 3] * ct[c + 3];
      }
      for (; c < dk; ++c) d0 += qh[c] * ct[c];
      sp_[h * tt + t] = (d0 + d1) + (d2 + d3);
    }
    __syncthreads();
    for (int h = tid >> 5; h < nh; h += kLatThreads / 32) {  // one warp per head
      const int lane = tid & 31;
      float mx = -INFINITY;
      for (int t = lane; t < cnt; t += 32) mx = fmaxf(mx, sp_[h * tt + t]);
      mx = fmaxf(warp_max(mx), sm[h]);
      float sum = 0.f;
      for (int t = lane; t < cnt; t += 32) {
        const float p = exp2f(sp_[h * tt + t] - mx);
        sp_[h * tt + t] = p;
        sum += p;
      }
      sum = warp_sum(sum);
      const float alpha = exp2f(sm[h] - mx);
      __syncwarp();
      if (lane == 0) {
        sm[h] = mx;
        sm[hg + h] = sm[hg + h] * alpha + sum;
        sm[2 * hg + h] = alpha;
      }
    }
    __syncthreads();
    for (int i = tid; i < nh * dv; i += kLatThreads) {
      const int h = i / dv, c = i - h * dv;
      float acc = so[i] * sm[2 * hg + h];
      for (int t = 0; t < cnt; ++t) acc += sp_[h * tt + t] * sv[t * ldv + c];
      so[i] = acc;
    }
  }
  __syncthreads();
  const long long RH = (long long)a.n_seq * a.Tn * a.H;
  for (int i = tid; i < nh * dv; i += kLatThreads) {
    const int h = i / dv, c = i - h * dv;
    const long long rh = (long long)row * a.H + h0 + h;
    const float sum = sm[hg + h];
    if (a.n_splits > 1) {
      const long long slot = (long long)split * RH + rh;
      a.ws_o[slot * dv + c] = so[i];
      if (c == 0) {
        a.ws_ml[2 * slot] = sm[h];
        a.ws_ml[2 * slot + 1] = sum;
      }
    } else {
      float f = sum > 0.f ? 1.f / sum : 0.f;
      if (a.gate) f *= 1.f / (1.f + expf(-Io<T>::ld(static_cast<const T*>(a.gate) + (long long)row * a.gate_rs + h0 + h)));
      Io<T>::st(static_cast<T*>(a.out) + (long long)row * a.out_rs + (long long)(h0 + h) * dv + c, so[i] * f);
    }
  }
}

// CTA per (row, head): the splits' weights once in shared memory, then one thread per column.
constexpr int kLatMaxSplits = 256;
template <typename T>
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentArgs a) {
  __shared__ float wt[kLatMaxSplits];
  __shared__ float scratch[40];
  const long long RH = (long long)a.n_seq * a.Tn * a.H;
  const long long rh = blockIdx.x;
  const long long row = rh / a.H;
  const int h = (int)(rh - row * a.H), tid = threadIdx.x, n = a.n_splits;
  float m = -INFINITY;
  for (int s = tid & 31; s < n; s += 32) m = fmaxf(m, a.ws_ml[2 * (s * RH + rh)]);
  m = warp_max(m);  // the same in every warp
  float l = 0.f;
  for (int s = tid; s < n; s += 128) {
    const float ms = a.ws_ml[2 * (s * RH + rh)];
    const float e = ms == -INFINITY ? 0.f : exp2f(ms - m);
    wt[s] = e;
    l += e == 0.f ? 0.f : a.ws_ml[2 * (s * RH + rh) + 1] * e;
  }
  l = block_sum(l, scratch);  // and `wt` is complete
  float f = l > 0.f ? 1.f / l : 0.f;
  if (a.gate) f *= 1.f / (1.f + expf(-Io<T>::ld(static_cast<const T*>(a.gate) + row * a.gate_rs + h)));
  T* dst = static_cast<T*>(a.out) + row * a.out_rs + (long long)h * a.dv;
  for (int c = tid; c < a.dv; c += 128) {
    float acc = 0.f;
    int s = 0;
    for (; s + 8 <= n; s += 8) {  // eight loads in flight; a split without keys has weight 0 and holds nothing
      float v[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) v[u] = a.ws_o[((s + u) * RH + rh) * a.dv + c];
#pragma unroll
      for (int u = 0; u < 8; ++u) acc += wt[s + u] == 0.f ? 0.f : wt[s + u] * v[u];
    }
    for (; s < n; ++s) acc += wt[s] == 0.f ? 0.f : wt[s] * a.ws_o[(s * RH + rh) * a.dv + c];
    Io<T>::st(dst + c, acc * f);
  }
}

static int latent_max_smem() {
  static int bytes[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return 0;
  if (bytes[dev] == 0) cudaDeviceGetAttribute(&bytes[dev], cudaDevAttrMaxSharedMemoryPerBlockOptin, dev);
  return bytes[dev];
}

template <typename T>
static int latent_simt_launch(const LatentArgs& a, cudaStream_t st) {
  const int limit = latent_max_smem();
  const int per = a.H / a.G;
  auto need = [&](int hg, int tt) {
    return ((size_t)hg * (a.dk + a.dv) + (size_t)tt * (a.dk + 1 + (a.v_col ? a.dv + 1 : 0)) + (size_t)hg * tt + 3 * hg) * 4;
  };
  int hg = per < 16 ? per : 16, tt = 32;
  while (need(hg, tt) > (size_t)limit && (hg > 1 || tt > 1)) {
    if (hg > 4 || (tt == 1 && hg > 1)) hg = (hg + 1) / 2;
    else tt = tt / 2;
  }
  const size_t smem = need(hg, tt);
  if (smem > (size_t)limit) {
    set_error("latent_attn: key size %d and value size %d do not fit the shared memory", a.dk, a.dv);
    return DGPT_E_UNSUPPORTED;
  }
  cudaError_t e = cudaFuncSetAttribute(latent_attn_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) {
    set_error("latent_attn: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
    return DGPT_E_CUDA;
  }
  const dim3 grid((unsigned)(a.n_seq * a.Tn), (unsigned)a.n_splits, (unsigned)(a.G * ((per + hg - 1) / hg)));
  latent_attn_kernel<T><<<grid, kLatThreads, smem, st>>>(a, hg, tt);
  return launch_status("latent_attn");
}

}  // namespace dgpt

using namespace dgpt;

extern "C" int dgpt_latent_append(const void* in, int64_t in_row_stride, const float* w, float eps, int32_t r_norm,
                                  const dgpt_kv_layout* kv, const int32_t* seq_slot0, const int32_t* step_ptr, int32_t n_seq,
                                  int32_t T, int32_t r, void* flat, int32_t dtype, int32_t* status, void* stream) {
  DGPT_REQUIRE(in && w && seq_slot0, "latent_append: NULL pointer");
  DGPT_REQUIRE(n_seq >= 0 && T >= 0 && r > 0 && r % 8 == 0 && r_norm > 0 && r_norm <= r,
               "latent_append: r must be a multiple of 8 that holds the %d normalised columns", r_norm);
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, "latent_append: unknown dtype %d", dtype);
  if (int e = validate_kv(kv, r)) return e;
  const long long n = (long long)n_seq * T;
  if (n == 0) return DGPT_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const unsigned grid = (unsigned)((n + 7) / 8);
  const KvView view = make_view(kv);
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const int vec = dtype == DGPT_F32 ? 4 : 8;
  const bool wide = r == r_norm && in_row_stride % vec == 0 && al16(in) && al16(w) && al16(flat) && kv->page_stride % vec == 0;
  const int nv = wide ? (r / vec + 31) / 32 : 0;
#define DGPT_LA(TT, NV)                                                                                                          \
  latent_append_kernel<TT, NV><<<grid, 256, 0, st>>>(static_cast<const TT*>(in), in_row_stride, w, eps, r_norm, view, seq_slot0, \
                                                     step_ptr, n_seq, T, r, static_cast<TT*>(flat), status)
#define DGPT_LAT(TT)                    \
  do {                                  \
    if (nv == 1) DGPT_LA(TT, 1);        \
    else if (nv == 2) DGPT_LA(TT, 2);   \
    else if (nv == 3 || nv == 4) DGPT_LA(TT, 4); \
    else DGPT_LA(TT, 0);                \
  } while (0)
  if (dtype == DGPT_F32) DGPT_LAT(float);
  else DGPT_LAT(__nv_bfloat16);
#undef DGPT_LAT
#undef DGPT_LA
  return launch_status("latent_append");
}

extern "C" size_t dgpt_latent_attn_workspace_bytes(int32_t R, int32_t H, int32_t r, int32_t n_splits) {
  if (n_splits <= 1) return 0;
  return (((size_t)R * H * n_splits * (size_t)(r + 2) * sizeof(float)) + 15) & ~(size_t)15;
}

// Checks, the choice of kernel and the merge of splits for both entry points.
static int row_attn(const char* what, const void* q, int64_t q_row_stride, const dgpt_kv_layout* kv, int32_t row_w, int32_t v_col,
                    const int32_t* len0, const int32_t* start1, const int32_t* len1, const int32_t* step_ptr, const void* gate,
                    int64_t gate_row_stride, void* out, int64_t out_row_stride, void* workspace, size_t workspace_bytes,
                    int32_t n_splits, int32_t n_seq, int32_t T, int32_t H, int32_t G, int32_t dk, int32_t dv, int32_t window,
                    int32_t keep_first, float scale, int32_t dtype, int32_t impl, int32_t* status, void* stream) {
  DGPT_REQUIRE(q && out && start1 && len1, "%s: NULL pointer", what);
  DGPT_REQUIRE(n_seq >= 0 && T >= 0 && H > 0 && G > 0 && H % G == 0 && dk > 0 && dk % 8 == 0 && dv > 0 && dv % 8 == 0 && window >= 0 &&
                   keep_first >= 0,
               "%s: bad sizes", what);
  DGPT_REQUIRE(row_w % 8 == 0 && v_col % 8 == 0 && row_w >= G * dk && (v_col == 0 ? dk == dv && G == 1 : v_col >= G * dk && row_w >= v_col + G * dv),
               "%s: keys and values do not fit a cache row of %d", what, row_w);
  DGPT_REQUIRE(n_splits >= 1 && n_splits <= kLatMaxSplits && H <= 65535, "%s: 1 to %d splits", what, kLatMaxSplits);
  DGPT_REQUIRE(impl >= 0 && impl <= 2, "%s: impl must be 0 (auto), 1 (CUDA cores) or 2 (tcgen05)", what);
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, "%s: unknown dtype %d", what, dtype);
  DGPT_REQUIRE((reinterpret_cast<uintptr_t>(q) & 15) == 0 && q_row_stride % 8 == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0 &&
                   out_row_stride % 8 == 0,
               "%s: q and out must be 16-byte aligned with row strides of a multiple of 8", what);
  if (int e = validate_kv(kv, row_w)) return e;
  const long long R = (long long)n_seq * T;
  if (R == 0) return DGPT_OK;
  DGPT_REQUIRE(R <= 0x7fffffff, "%s: too many rows", what);
  const size_t need = dgpt_latent_attn_workspace_bytes((int32_t)R, H, dv, n_splits);
  if (need > 0 && (workspace == nullptr || workspace_bytes < need || (reinterpret_cast<uintptr_t>(workspace) & 15) != 0)) {
    set_error("%s: a 16-byte aligned workspace of %zu bytes is needed, %zu given", what, need, workspace_bytes);
    return DGPT_E_WORKSPACE;
  }
  LatentArgs a;
  a.q = q; a.q_rs = q_row_stride;
  a.kv = make_view(kv);
  a.len0 = len0; a.start1 = start1; a.len1 = len1; a.step_ptr = step_ptr;
  a.gate = gate; a.gate_rs = gate_row_stride;
  a.out = out; a.out_rs = out_row_stride;
  a.ws_o = static_cast<float*>(workspace);
  a.ws_ml = workspace ? a.ws_o + (size_t)R * H * n_splits * dv : nullptr;
  a.n_splits = n_splits; a.n_seq = n_seq; a.Tn = T; a.H = H; a.window = window;
  a.G = G; a.dk = dk; a.dv = dv; a.row_w = row_w; a.v_col = v_col; a.keep = keep_first;
  a.scale_log2 = scale * kLog2e;
  a.status = status;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool tc_ok = latent_tc_supported(a, *kv, dtype);
  if (impl == 2 && !tc_ok) {
    set_error("%s: the tcgen05 kernel covers bf16 with key and value sizes up to 512 in dense runs or pages that tile 128 keys "
              "(sizes %d and %d, dtype %d, page_tokens %d)", what, dk, dv, dtype, kv->page_tokens);
    return DGPT_E_UNSUPPORTED;
  }
  int e;
  if (tc_ok && impl != 1) e = latent_tc_launch(a, *kv, st);
  else if (dtype == DGPT_F32) e = latent_simt_launch<float>(a, st);
  else e = latent_simt_launch<__nv_bfloat16>(a, st);
  if (e || n_splits == 1) return e;
  const long long RH = R * H;
  if (dtype == DGPT_F32) latent_combine_kernel<float><<<(unsigned)RH, 128, 0, st>>>(a);
  else latent_combine_kernel<__nv_bfloat16><<<(unsigned)RH, 128, 0, st>>>(a);
  return launch_status("latent_combine");
}

extern "C" int dgpt_latent_attn(const void* q, int64_t q_row_stride, const dgpt_kv_layout* kv, const int32_t* len0,
                                const int32_t* start1, const int32_t* len1, const int32_t* step_ptr, const void* gate,
                                int64_t gate_row_stride, void* out, int64_t out_row_stride, void* workspace,
                                size_t workspace_bytes, int32_t n_splits, int32_t n_seq, int32_t T, int32_t H, int32_t r,
                                int32_t window, float scale, int32_t dtype, int32_t impl, int32_t* status, void* stream) {
  return row_attn("latent_attn", q, q_row_stride, kv, r, 0, len0, start1, len1, step_ptr, gate, gate_row_stride, out, out_row_stride,
                  workspace, workspace_bytes, n_splits, n_seq, T, H, 1, r, r, window, 0, scale, dtype, impl, status, stream);
}

extern "C" int dgpt_grouped_attn(const void* q, int64_t q_row_stride, const dgpt_kv_layout* kv, int32_t row_width, int32_t v_col,
                                 const int32_t* len0, const int32_t* start1, const int32_t* len1, const int32_t* step_ptr,
                                 const void* gate, int64_t gate_row_stride, void* out, int64_t out_row_stride, void* workspace,
                                 size_t workspace_bytes, int32_t n_splits, int32_t n_seq, int32_t T, int32_t H, int32_t G,
                                 int32_t dk, int32_t dv, int32_t window, int32_t keep_first, float scale, int32_t dtype,
                                 int32_t impl, int32_t* status, void* stream) {
  DGPT_REQUIRE(v_col > 0, "grouped_attn: the values follow the keys in a cache row");
  return row_attn("grouped_attn", q, q_row_stride, kv, row_width, v_col, len0, start1, len1, step_ptr, gate, gate_row_stride, out,
                  out_row_stride, workspace, workspace_bytes, n_splits, n_seq, T, H, G, dk, dv, window, keep_first, scale, dtype, impl,
                  status, stream);
}
