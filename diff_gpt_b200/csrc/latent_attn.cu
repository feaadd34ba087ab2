// Attention over a cache of latents (one vector of r numbers per token, shared by all heads) with the key and value
// expansions absorbed into the query and the output: q~_h = W_uk,h^T q_h and o_h = W_uv,h (sum_j p_j c_j), so scores and
// sums are formed on the latents themselves and the cache is read once for all heads.  A sliding window limits which
// latents a query sees.
//
//   latent_append_kernel   c = rms_norm(x) * w, rounded once, into the paged cache (and a flat copy where asked for)
//   latent_attn_mma_kernel bf16, r <= 512: CTA per (query, key split, group of 16 heads).  Decode reads
//                          window * r * 2 bytes per query whatever the number of heads, i.e. it is HBM-bound up to
//                          about 16 heads; the 16 x 64 x r products of a tile run on mma.sync (M = 16 heads: a
//                          tcgen05 tile would be 7/8 padding)
//   latent_attn_kernel     any r and storage type (fp32 models): scores and sums in fp32 on the CUDA cores
//   latent_combine_kernel  merges key splits
// Keys of sequence s, token t of the call: logical keys [0, n) with n = len0[s] + len1[s] + step + t, where logical key i
// is slot i below len0 and slot start1 + (i - len0) above; the query sees the last `window` of them (0 = all).
#include "common.cuh"

namespace dgpt {

constexpr int kLatTile = 64;      // keys per tile of the mma kernel
constexpr int kLatThreads = 256;  // 8 warps
constexpr int kLatHeads = 16;     // heads per CTA (the M of mma.m16n8k16)

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
};

// which logical keys a (row, split) covers and how they map to slots
struct LatentSpan {
  int seq, n0, s1, begin, end;
};
__device__ __forceinline__ LatentSpan latent_span(const LatentArgs& a, int row, int split, int tile) {
  LatentSpan sp;
  sp.seq = row / a.Tn;
  const int t = row - sp.seq * a.Tn;
  const int cap = a.kv.page_table ? a.kv.max_pages * a.kv.page_tokens : a.kv.page_tokens;
  sp.n0 = a.len0 ? min(max(a.len0[sp.seq], 0), cap) : 0;
  sp.s1 = min(max(a.start1[sp.seq], 0), cap);
  const int n1 = a.len1[sp.seq] + (a.step_ptr ? *a.step_ptr : 0) + t;
  const int n = sp.n0 + min(max(n1, 0), cap - sp.s1);  // never past the sequence's slots
  const int lo = a.window > 0 ? max(0, n - a.window) : 0;
  int chunk = (n - lo + a.n_splits - 1) / a.n_splits;
  chunk = (chunk + tile - 1) / tile * tile;
  sp.begin = lo + split * chunk;
  sp.end = min(n, sp.begin + chunk);
  return sp;
}
// Element offset of logical key i, or -1 when its table entry lies outside the pool.
__device__ __forceinline__ long long latent_offset(const LatentArgs& a, const LatentSpan& sp, int i) {
  const int slot = i < sp.n0 ? i : sp.s1 + (i - sp.n0);
  const int lp = slot / a.kv.page_tokens;
  const int in = slot - lp * a.kv.page_tokens;
  long long pg = sp.seq;
  if (a.kv.page_table) {
    pg = a.kv.page_table[(long long)sp.seq * a.kv.max_pages + lp];
    if (a.kv.n_pages > 0 && (pg < 0 || pg >= a.kv.n_pages)) return -1;
  }
  return pg * a.kv.page_stride + (long long)in * a.r;
}

// ---- append ---------------------------------------------------------------------------------
template <typename T>
__global__ void latent_append_kernel(const T* __restrict__ in, long long in_rs, const float* __restrict__ w, float eps, int r_norm,
                                     KvView kv, const int* __restrict__ slot0, const int* __restrict__ step_ptr, int n_seq, int Tn,
                                     int r, T* __restrict__ flat, int* status) {
  const long long tok = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (tok >= (long long)n_seq * Tn) return;
  const int lane = threadIdx.x & 31;
  const int s = (int)(tok / Tn), t = (int)(tok - (long long)s * Tn);
  const T* x = in + tok * in_rs;
  float ss = 0.f;
  for (int c = lane; c < r_norm; c += 32) {
    const float v = Io<T>::ld(x + c);
    ss += v * v;
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
  for (int c = lane; c < r; c += 32) {
    const float v = c < r_norm ? Io<T>::ld(x + c) * inv * w[c] : 0.f;
    if (dst) Io<T>::st(dst + c, v);
    if (flat) Io<T>::st(flat + tok * r + c, v);
  }
}

// ---- bf16 on mma.sync ---------------------------------------------------------------------------
__device__ __forceinline__ uint32_t lat_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;  // 0 source bytes: the destination is filled with zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}

// Row stride (elements) of a latent in shared memory: r rounded up to a k-step of 16, plus 16 bytes - an odd number of
// 16-byte units, so that the eight rows of an ldmatrix fall into different banks.
__host__ __device__ inline int lat_ld(int r) { return (r + 15) / 16 * 16 + 8; }
constexpr int kLatPLd = kLatTile + 8;
inline size_t lat_smem_bytes(int r, int stages) {
  return (size_t)(kLatHeads + stages * kLatTile) * lat_ld(r) * 2 + (size_t)kLatHeads * kLatPLd * 2 +
         8 * kLatHeads * 4 * 2 + 8 * 32 * 4 * 4;
}

// NT = 8-column groups of the output per warp (8 NT columns, 64 NT in all: r <= 64 NT).
// Scores: warp = (16-key group tg, half kh of the r columns); the two halves swap partial sums so that each warp ends up
// with the 16 heads x 8 keys block (tg, kh).  Sums: warp w owns columns [8 NT w, 8 NT (w + 1)) for all 64 keys.
template <int NT>
__global__ void __launch_bounds__(kLatThreads, NT <= 2 ? 3 : 1) latent_attn_mma_kernel(const LatentArgs a, int stages) {
  using B16 = __nv_bfloat16;
  extern __shared__ __align__(16) uint8_t lat_raw[];
  const int ld = lat_ld(a.r);
  B16* sQ = reinterpret_cast<B16*>(lat_raw);
  B16* sC = sQ + kLatHeads * ld;
  B16* sP = sC + (size_t)stages * kLatTile * ld;
  float* sMax = reinterpret_cast<float*>(sP + kLatHeads * kLatPLd);  // [8][16]
  float* sSum = sMax + 8 * kLatHeads;                                // [8][16]
  float* sX = sSum + 8 * kLatHeads;                                  // [8 warps][32 lanes][4]: partial scores to swap
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row = blockIdx.x, split = blockIdx.y, h0 = blockIdx.z * kLatHeads;
  const LatentSpan sp = latent_span(a, row, split, kLatTile);
  const int n_tiles = sp.end > sp.begin ? (sp.end - sp.begin + kLatTile - 1) / kLatTile : 0;
  const int cpr = a.r / 8;  // 16-byte chunks per latent (r is a multiple of 8)
  const B16* pool = static_cast<const B16*>(a.kv.k);

  // columns [r, ld) of every row are read by the last k-step and never loaded: clear them once
  const int tail = ld - a.r;
  for (int i = tid; i < (kLatHeads + stages * kLatTile) * tail; i += kLatThreads)
    sQ[(size_t)(i / tail) * ld + a.r + i % tail] = __float2bfloat16_rn(0.f);
  for (int i = tid; i < kLatHeads * cpr; i += kLatThreads) {
    const int h = i / cpr, c = (i - h * cpr) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (h0 + h < a.H)
      v = *reinterpret_cast<const uint4*>(static_cast<const B16*>(a.q) + (long long)row * a.q_rs + (long long)(h0 + h) * a.r + c);
    *reinterpret_cast<uint4*>(sQ + (size_t)h * ld + c) = v;
  }

  // loader: this thread's chunks of a tile are (tok, ch), (tok + d_tok, ch + d_ch), ...
  const int tok0 = tid / cpr, ch0 = tid - tok0 * cpr, d_tok = kLatThreads / cpr, d_ch = kLatThreads - d_tok * cpr;
  auto load_tile = [&](int tile) {
    if (tile < n_tiles) {
      const int i0 = sp.begin + tile * kLatTile;
      B16* dst = sC + (size_t)(tile % stages) * kLatTile * ld;
      int tok = tok0, ch = ch0;
      while (tok < kLatTile) {
        const int i = i0 + tok;
        long long off = -1;
        if (i < sp.end) off = latent_offset(a, sp, i);
        cp_async16(lat_smem(dst + (size_t)tok * ld + ch * 8), pool + (off < 0 ? 0 : off + ch * 8), off >= 0);
        tok += d_tok;
        ch += d_ch;
        if (ch >= cpr) {
          ch -= cpr;
          ++tok;
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");  // one group per tile, empty ones included
  };
  for (int s = 0; s < stages - 1; ++s) load_tile(s);
  __syncthreads();

  const int tg = warp >> 1, kh = warp & 1;
  const int ksteps = (a.r + 15) / 16, kmid = (ksteps + 1) / 2;
  const int k_begin = kh ? kmid : 0, k_n = kh ? ksteps - kmid : kmid;  // at most 2 NT steps
  uint32_t qf[2 * NT][4];
#pragma unroll
  for (int k = 0; k < 2 * NT; ++k) {
    if (k < k_n)
      ldsm4(lat_smem(sQ + (size_t)((lane >> 3 & 1) * 8 + (lane & 7)) * ld + (k_begin + k) * 16 + (lane >> 4) * 8), qf[k]);
  }
  float o[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const int hr = lane >> 2;  // this thread's head rows: hr and hr + 8
  const int col0 = warp * NT * 8;

  for (int tile = 0; tile < n_tiles; ++tile) {
    if (stages == 2) asm volatile("cp.async.wait_group 0;" ::: "memory");
    else if (stages == 3) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else asm volatile("cp.async.wait_group 2;" ::: "memory");
    __syncthreads();  // the tile is visible to all warps, and everybody has left the one before
    load_tile(tile + stages - 1);
    const B16* c = sC + (size_t)(tile % stages) * kLatTile * ld;
    // ---- scores of 16 heads x 16 keys over this warp's half of the columns ----
    float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
    const uint32_t cb = lat_smem(c + (size_t)(tg * 16 + (lane >> 4) * 8 + (lane & 7)) * ld + (lane >> 3 & 1) * 8);
#pragma unroll
    for (int k = 0; k < 2 * NT; ++k) {
      if (k < k_n) {
        uint32_t b[4];
        ldsm4(cb + (k_begin + k) * 32, b);
        mma16816(s0, qf[k], b[0], b[1]);
        mma16816(s1, qf[k], b[2], b[3]);
      }
    }
    // swap: the half kh keeps key block kh
    float4* mine = reinterpret_cast<float4*>(sX + (warp * 32 + lane) * 4);
    *mine = kh ? make_float4(s0[0], s0[1], s0[2], s0[3]) : make_float4(s1[0], s1[1], s1[2], s1[3]);
    asm volatile("bar.sync %0, 64;" ::"r"(1 + tg) : "memory");
    const float4 theirs = *reinterpret_cast<const float4*>(sX + ((warp ^ 1) * 32 + lane) * 4);
    float s[4];
    s[0] = (kh ? s1[0] : s0[0]) + theirs.x;
    s[1] = (kh ? s1[1] : s0[1]) + theirs.y;
    s[2] = (kh ? s1[2] : s0[2]) + theirs.z;
    s[3] = (kh ? s1[3] : s0[3]) + theirs.w;
    const int kcol = tg * 16 + kh * 8 + (lane & 3) * 2;
    const int left = sp.end - sp.begin - tile * kLatTile;
#pragma unroll
    for (int e = 0; e < 4; ++e) s[e] = kcol + (e & 1) < left ? s[e] * a.scale_log2 : -INFINITY;
    float mx[2] = {fmaxf(s[0], s[1]), fmaxf(s[2], s[3])};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
    }
    if ((lane & 3) == 0) {
      sMax[warp * kLatHeads + hr] = mx[0];
      sMax[warp * kLatHeads + hr + 8] = mx[1];
    }
    __syncthreads();
    float alpha[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float mn = m[e];
#pragma unroll
      for (int w = 0; w < 8; ++w) mn = fmaxf(mn, sMax[w * kLatHeads + hr + 8 * e]);
      alpha[e] = exp2f(m[e] - mn);  // the first key of a tile is always there, so mn is finite
      m[e] = mn;
    }
    const float p0 = exp2f(s[0] - m[0]), p1 = exp2f(s[1] - m[0]), p2 = exp2f(s[2] - m[1]), p3 = exp2f(s[3] - m[1]);
    l[0] = l[0] * alpha[0] + (p0 + p1);
    l[1] = l[1] * alpha[1] + (p2 + p3);
    *reinterpret_cast<__nv_bfloat162*>(sP + hr * kLatPLd + kcol) = __floats2bfloat162_rn(p0, p1);
    *reinterpret_cast<__nv_bfloat162*>(sP + (hr + 8) * kLatPLd + kcol) = __floats2bfloat162_rn(p2, p3);
    __syncthreads();
    // ---- o += P C over this warp's columns ----
    if (col0 < a.r) {
      if (alpha[0] != 1.f || alpha[1] != 1.f) {
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          o[i][0] *= alpha[0];
          o[i][1] *= alpha[0];
          o[i][2] *= alpha[1];
          o[i][3] *= alpha[1];
        }
      }
#pragma unroll
      for (int kk = 0; kk < kLatTile / 16; ++kk) {
        uint32_t pf[4];
        ldsm4(lat_smem(sP + (size_t)((lane >> 3 & 1) * 8 + (lane & 7)) * kLatPLd + kk * 16 + (lane >> 4) * 8), pf);
        const uint32_t vb = lat_smem(c + (size_t)(kk * 16 + (lane >> 3 & 1) * 8 + (lane & 7)) * ld + col0 + (lane >> 4) * 8);
#pragma unroll
        for (int i = 0; i < NT; i += 2) {
          if (col0 + i * 8 < a.r) {  // warp-uniform; the pair's second half may be the cleared padding
            uint32_t b[4];
            ldsm4_t(vb + i * 16, b);
            mma16816(o[i], pf, b[0], b[1]);
            mma16816(o[i + 1], pf, b[2], b[3]);
          }
        }
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  // ---- row sums over the four lanes of a row and the eight warps ----
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
  }
  if ((lane & 3) == 0) {
    sSum[warp * kLatHeads + hr] = l[0];
    sSum[warp * kLatHeads + hr + 8] = l[1];
  }
  __syncthreads();
  const long long RH = (long long)a.n_seq * a.Tn * a.H;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int h = h0 + hr + 8 * e;
    if (h >= a.H) continue;
    float sum = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) sum += sSum[w * kLatHeads + hr + 8 * e];
    const long long rh = (long long)row * a.H + h;
    if (a.n_splits > 1) {
      const long long slot = (long long)split * RH + rh;
      if (warp == 0 && (lane & 3) == 0) {
        a.ws_ml[2 * slot] = m[e];
        a.ws_ml[2 * slot + 1] = sum;
      }
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int c = col0 + i * 8 + (lane & 3) * 2;
        if (c < a.r) *reinterpret_cast<float2*>(a.ws_o + slot * a.r + c) = make_float2(o[i][2 * e], o[i][2 * e + 1]);
      }
    } else {
      float f = sum > 0.f ? 1.f / sum : 0.f;
      if (a.gate) f *= 1.f / (1.f + __expf(-__bfloat162float(static_cast<const B16*>(a.gate)[(long long)row * a.gate_rs + h])));
      B16* dst = static_cast<B16*>(a.out) + (long long)row * a.out_rs + (long long)h * a.r;
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int c = col0 + i * 8 + (lane & 3) * 2;
        if (c < a.r) *reinterpret_cast<__nv_bfloat162*>(dst + c) = __floats2bfloat162_rn(o[i][2 * e] * f, o[i][2 * e + 1] * f);
      }
    }
  }
}

// ---- any r, any storage type, CUDA cores -------------------------------------------------------
// Shared memory: q and o of `hg` heads in fp32, a tile of `tt` latents in fp32 (row stride r + 1), scores.
template <typename T>
__global__ void __launch_bounds__(kLatThreads) latent_attn_kernel(const LatentArgs a, int hg, int tt) {
  extern __shared__ __align__(16) uint8_t lat_raw[];
  const int r = a.r, ldc = r + 1;
  float* sq = reinterpret_cast<float*>(lat_raw);  // [hg][r]
  float* so = sq + hg * r;                        // [hg][r]
  float* sc = so + hg * r;                        // [tt][r + 1]
  float* sp_ = sc + tt * ldc;                     // [hg][tt]
  float* sm = sp_ + hg * tt;                      // [hg] running maximum, [hg] sum, [hg] rescale
  const int tid = threadIdx.x;
  const int row = blockIdx.x, split = blockIdx.y, h0 = blockIdx.z * hg;
  const int nh = min(hg, a.H - h0);
  const LatentSpan sp = latent_span(a, row, split, 32);
  const T* q = static_cast<const T*>(a.q) + (long long)row * a.q_rs + (long long)h0 * r;
  for (int i = tid; i < nh * r; i += kLatThreads) {
    sq[i] = Io<T>::ld(q + i) * a.scale_log2;
    so[i] = 0.f;
  }
  if (tid < nh) {
    sm[tid] = -INFINITY;
    sm[hg + tid] = 0.f;
  }
  const T* pool = static_cast<const T*>(a.kv.k);
  for (int i0 = sp.begin; i0 < sp.end; i0 += tt) {
    const int cnt = min(tt, sp.end - i0);
    __syncthreads();
    for (int t = tid >> 5; t < cnt; t += kLatThreads / 32) {
      const long long off = latent_offset(a, sp, i0 + t);
      for (int c = tid & 31; c < r; c += 32) sc[t * ldc + c] = off < 0 ? 0.f : Io<T>::ld(pool + off + c);
    }
    __syncthreads();
    for (int i = tid; i < nh * cnt; i += kLatThreads) {
      const int h = i / cnt, t = i - h * cnt;
      const float* qh = sq + h * r;
      const float* ct = sc + t * ldc;
      float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
      int c = 0;
      for (; c + 4 <= r; c += 4) {
        d0 += qh[c] * ct[c];
        d1 += qh[c + 1] * ct[c + 1];
        d2 += qh[c + 2] * ct[c + 2];
        d3 += qh[c + 3] * ct[c + 3];
      }
      for (; c < r; ++c) d0 += qh[c] * ct[c];
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
    for (int i = tid; i < nh * r; i += kLatThreads) {
      const int h = i / r, c = i - h * r;
      float acc = so[i] * sm[2 * hg + h];
      for (int t = 0; t < cnt; ++t) acc += sp_[h * tt + t] * sc[t * ldc + c];
      so[i] = acc;
    }
  }
  __syncthreads();
  const long long RH = (long long)a.n_seq * a.Tn * a.H;
  for (int i = tid; i < nh * r; i += kLatThreads) {
    const int h = i / r, c = i - h * r;
    const long long rh = (long long)row * a.H + h0 + h;
    const float sum = sm[hg + h];
    if (a.n_splits > 1) {
      const long long slot = (long long)split * RH + rh;
      a.ws_o[slot * r + c] = so[i];
      if (c == 0) {
        a.ws_ml[2 * slot] = sm[h];
        a.ws_ml[2 * slot + 1] = sum;
      }
    } else {
      float f = sum > 0.f ? 1.f / sum : 0.f;
      if (a.gate) f *= 1.f / (1.f + expf(-Io<T>::ld(static_cast<const T*>(a.gate) + (long long)row * a.gate_rs + h0 + h)));
      Io<T>::st(static_cast<T*>(a.out) + (long long)row * a.out_rs + (long long)(h0 + h) * r + c, so[i] * f);
    }
  }
}

// One warp per (row, head): every lane knows the weights of all splits, then the columns are summed over the splits.
template <typename T>
__global__ void latent_combine_kernel(const LatentArgs a) {
  const long long RH = (long long)a.n_seq * a.Tn * a.H;
  const long long rh = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (rh >= RH) return;
  const int lane = threadIdx.x & 31;
  const long long row = rh / a.H;
  const int h = (int)(rh - row * a.H);
  float m = -INFINITY;
  for (int s = lane; s < a.n_splits; s += 32) m = fmaxf(m, a.ws_ml[2 * (s * RH + rh)]);
  m = warp_max(m);
  float l = 0.f;
  for (int s = lane; s < a.n_splits; s += 32) {
    const float ms = a.ws_ml[2 * (s * RH + rh)];
    l += ms == -INFINITY ? 0.f : a.ws_ml[2 * (s * RH + rh) + 1] * exp2f(ms - m);
  }
  l = warp_sum(l);
  float f = l > 0.f ? 1.f / l : 0.f;
  if (a.gate) f *= 1.f / (1.f + expf(-Io<T>::ld(static_cast<const T*>(a.gate) + row * a.gate_rs + h)));
  T* dst = static_cast<T*>(a.out) + row * a.out_rs + (long long)h * a.r;
  for (int c = lane; c < a.r; c += 32) {
    float acc = 0.f;
    for (int s = 0; s < a.n_splits; ++s) {
      const float ms = a.ws_ml[2 * (s * RH + rh)];
      if (ms != -INFINITY) acc += a.ws_o[(s * RH + rh) * a.r + c] * exp2f(ms - m);
    }
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

template <int NT>
static int latent_mma_launch(const LatentArgs& a, cudaStream_t st) {
  const int limit = latent_max_smem();
  // as many tiles in flight as fit: three where the SM holds more than one CTA, else up to four
  int stages = NT <= 2 ? 3 : 4;
  while (stages > 2 && lat_smem_bytes(a.r, stages) > (size_t)limit) --stages;
  const size_t smem = lat_smem_bytes(a.r, stages);
  if (smem > (size_t)limit) {
    set_error("latent_attn: r = %d does not fit the shared memory", a.r);
    return DGPT_E_UNSUPPORTED;
  }
  cudaError_t e = cudaFuncSetAttribute(latent_attn_mma_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) {
    set_error("latent_attn: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
    return DGPT_E_CUDA;
  }
  const dim3 grid((unsigned)(a.n_seq * a.Tn), (unsigned)a.n_splits, (unsigned)((a.H + kLatHeads - 1) / kLatHeads));
  latent_attn_mma_kernel<NT><<<grid, kLatThreads, smem, st>>>(a, stages);
  return launch_status("latent_attn");
}

template <typename T>
static int latent_simt_launch(const LatentArgs& a, cudaStream_t st) {
  const int limit = latent_max_smem();
  auto need = [&](int hg, int tt) { return ((size_t)2 * hg * a.r + (size_t)tt * (a.r + 1) + (size_t)hg * tt + 3 * hg) * 4; };
  int hg = a.H < 16 ? a.H : 16, tt = 32;
  while (need(hg, tt) > (size_t)limit && (hg > 1 || tt > 1)) {
    if (hg > 4 || (tt == 1 && hg > 1)) hg = (hg + 1) / 2;
    else tt = tt / 2;
  }
  const size_t smem = need(hg, tt);
  if (smem > (size_t)limit) {
    set_error("latent_attn: r = %d does not fit the shared memory", a.r);
    return DGPT_E_UNSUPPORTED;
  }
  cudaError_t e = cudaFuncSetAttribute(latent_attn_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) {
    set_error("latent_attn: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
    return DGPT_E_CUDA;
  }
  const dim3 grid((unsigned)(a.n_seq * a.Tn), (unsigned)a.n_splits, (unsigned)((a.H + hg - 1) / hg));
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
  if (dtype == DGPT_F32)
    latent_append_kernel<float><<<grid, 256, 0, st>>>(static_cast<const float*>(in), in_row_stride, w, eps, r_norm, view, seq_slot0,
                                                      step_ptr, n_seq, T, r, static_cast<float*>(flat), status);
  else
    latent_append_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(static_cast<const __nv_bfloat16*>(in), in_row_stride, w, eps, r_norm,
                                                              view, seq_slot0, step_ptr, n_seq, T, r,
                                                              static_cast<__nv_bfloat16*>(flat), status);
  return launch_status("latent_append");
}

extern "C" size_t dgpt_latent_attn_workspace_bytes(int32_t R, int32_t H, int32_t r, int32_t n_splits) {
  if (n_splits <= 1) return 0;
  return (((size_t)R * H * n_splits * (size_t)(r + 2) * sizeof(float)) + 15) & ~(size_t)15;
}

extern "C" int dgpt_latent_attn(const void* q, int64_t q_row_stride, const dgpt_kv_layout* kv, const int32_t* len0,
                                const int32_t* start1, const int32_t* len1, const int32_t* step_ptr, const void* gate,
                                int64_t gate_row_stride, void* out, int64_t out_row_stride, void* workspace,
                                size_t workspace_bytes, int32_t n_splits, int32_t n_seq, int32_t T, int32_t H, int32_t r,
                                int32_t window, float scale, int32_t dtype, int32_t impl, void* stream) {
  DGPT_REQUIRE(q && out && start1 && len1, "latent_attn: NULL pointer");
  DGPT_REQUIRE(n_seq >= 0 && T >= 0 && H > 0 && r > 0 && r % 8 == 0 && window >= 0, "latent_attn: bad sizes");
  DGPT_REQUIRE(n_splits >= 1 && n_splits <= 65535 && H <= 65535, "latent_attn: bad number of splits or heads");
  DGPT_REQUIRE(impl >= 0 && impl <= 2, "latent_attn: impl must be 0 (auto), 1 (CUDA cores) or 2 (mma)");
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, "latent_attn: unknown dtype %d", dtype);
  DGPT_REQUIRE((reinterpret_cast<uintptr_t>(q) & 15) == 0 && q_row_stride % 8 == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0 &&
                   out_row_stride % 8 == 0,
               "latent_attn: q and out must be 16-byte aligned with row strides of a multiple of 8");
  if (int e = validate_kv(kv, r)) return e;
  const long long R = (long long)n_seq * T;
  if (R == 0) return DGPT_OK;
  DGPT_REQUIRE(R <= 0x7fffffff, "latent_attn: too many rows");
  const size_t need = dgpt_latent_attn_workspace_bytes((int32_t)R, H, r, n_splits);
  if (need > 0 && (workspace == nullptr || workspace_bytes < need || (reinterpret_cast<uintptr_t>(workspace) & 15) != 0)) {
    set_error("latent_attn: a 16-byte aligned workspace of %zu bytes is needed, %zu given", need, workspace_bytes);
    return DGPT_E_WORKSPACE;
  }
  LatentArgs a;
  a.q = q; a.q_rs = q_row_stride;
  a.kv = make_view(kv);
  a.len0 = len0; a.start1 = start1; a.len1 = len1; a.step_ptr = step_ptr;
  a.gate = gate; a.gate_rs = gate_row_stride;
  a.out = out; a.out_rs = out_row_stride;
  a.ws_o = static_cast<float*>(workspace);
  a.ws_ml = workspace ? a.ws_o + (size_t)R * H * n_splits * r : nullptr;
  a.n_splits = n_splits; a.n_seq = n_seq; a.Tn = T; a.H = H; a.r = r; a.window = window;
  a.scale_log2 = scale * kLog2e;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool mma_ok = dtype == DGPT_BF16 && r <= 512;
  if (impl == 2 && !mma_ok) {
    set_error("latent_attn: the mma kernel covers bf16 with r <= 512 (r = %d, dtype %d)", r, dtype);
    return DGPT_E_UNSUPPORTED;
  }
  int e;
  if (mma_ok && impl != 1) e = r <= 128 ? latent_mma_launch<2>(a, st) : (r <= 256 ? latent_mma_launch<4>(a, st) : latent_mma_launch<8>(a, st));
  else if (dtype == DGPT_F32) e = latent_simt_launch<float>(a, st);
  else e = latent_simt_launch<__nv_bfloat16>(a, st);
  if (e || n_splits == 1) return e;
  const long long RH = R * H;
  const unsigned grid = (unsigned)((RH + 7) / 8);
  if (dtype == DGPT_F32) latent_combine_kernel<float><<<grid, 256, 0, st>>>(a);
  else latent_combine_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(a);
  return launch_status("latent_combine");
}
