// Retention over many tokens on tcgen05 (sm_100a): the recurrence in chunks of up to 128 tokens.
//
// Inside a chunk of n tokens (i, j from 0), with S the fp32 state in front of it and the decays folded into the operands,
//   q^_i = decay^(i+1) q_i       k^_j = decay^(n-1-j) k_j
//   A    = q^ k^T                P_ij = decay^(-n) A_ij for j <= i, else 0          (= decay^(i-j) q_i . k_j)
//   o    = q^ S + P v            S <- decay^n S + k^^T v
// so every product is a plain matrix product into a TMEM accumulator, and no scale is applied after one.  q and k are
// rotated, scaled and decayed in fp32.  As operands all fp32 quantities (q^, k^, P, S) go in as two bf16 terms, high and
// low, whose products are summed in the fp32 accumulators (the product of two low terms is left out): about 17 significant
// bits; v is bf16 to begin with.  A chunk is shorter than 128 tokens where decay^(2n) would leave fp32's range.
//
// One CTA per (sequence, head, 128 value columns, segment of the tokens).  Few heads leave most SMs idle, so a long sequence
// is cut into segments: retention_state_kernel forms each segment's own contribution to the state, retention_prefix_kernel
// adds them up to the state behind each segment, and retention_tc_kernel starts every segment from there.
//   warps 0-15      rotate, split and write q^, k^ of a chunk into swizzled shared memory (v goes there by cp.async); A -> P;
//                   state -> shared memory; head norm, output gate and store.  Where every dimension is rotated the next
//                   chunk's q and k are fetched into registers while the products of this one run
//   warp 16         issues the products (one lane)
// TMEM columns: A [0, 128)  P high [128, 192)  P low [192, 256)  o [256, 384)  state [384, 512) (lane = key dimension).
// Every mbarrier wait is bounded; when one runs out the CTA leaves its loop together, gives what it issued a bounded chance to
// finish, frees TMEM and reports through the status word.
#include "retention.cuh"
#include "tcgen05.cuh"

namespace dgpt {
namespace tc {

constexpr int kRtWorkers = 512, kRtThreads = kRtWorkers + 32;  // sixteen worker warps, the MMA issuer's warp
constexpr long long kRtDrainCycles = 200000000ll;
constexpr int kRtChunk = 128;
constexpr uint32_t kRtBlock = 128 * 128;  // [128 rows][64 columns] bf16, swizzled
constexpr uint32_t kRtA = 0, kRtPh = 128, kRtPl = 192, kRtO = 256, kRtS = 384;

struct RtParams {
  RetentionArgs a;
  int n_seg, seg_len, n_slice;
  float* seg_state;  // [n_seq, H, n_seg - 1, dim, vdim]
};

__device__ __forceinline__ void rt_split2(uint64_t xy, uint32_t& hi, uint32_t& lo) {  // two packed fp32
  float x, y;
  unpack2(xy, x, y);
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const uint64_t neg = pack2(__uint_as_float((hi << 16) ^ 0x80000000u), __uint_as_float((hi & 0xffff0000u) ^ 0x80000000u));
  unpack2(add2(xy, neg), x, y);  // exact
  const __nv_bfloat162 l = __floats2bfloat162_rn(x, y);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ void rt_split(float x, float y, uint32_t& hi, uint32_t& lo) { rt_split2(pack2(x, y), hi, lo); }
// Eight columns from c on (a multiple of 8) of row r, as high and low terms `lo_off` bytes apart.
__device__ __forceinline__ void rt_store8(uint8_t* base, uint32_t lo_off, int r, int c, const float* v) {
  uint32_t h[4], l[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) rt_split(v[2 * i], v[2 * i + 1], h[i], l[i]);
  uint8_t* p = base + (c >> 6) * kRtBlock + r * 128 + ((((c & 63) >> 3) ^ (r & 7)) << 4);
  *reinterpret_cast<uint4*>(p) = make_uint4(h[0], h[1], h[2], h[3]);
  *reinterpret_cast<uint4*>(p + lo_off) = make_uint4(l[0], l[1], l[2], l[3]);
}
__device__ __forceinline__ float rt_pow(float l2, int n) { return n == 0 ? 1.f : exp2f((float)n * l2); }

// Columns [c, c + 8) of one rotated vector times f where they do not come as aligned pairs of eights: columns that pass
// unrotated (`passes`), or any columns, one by one; zeros from dim on.
__device__ __forceinline__ void rt_group(const RetentionArgs& a, bool passes, const __nv_bfloat16* x, const float2* cs, int c, float f,
                                         float* out) {
  const int half = a.rot >> 1;
  if (passes) {
    if (c < a.dim) ld16<__nv_bfloat16>(x + c, out);  // both are multiples of 8
#pragma unroll
    for (int e = 0; e < 8; ++e) out[e] *= f;
    return;
  }
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    const int d = c + e;
    float v = 0.f;
    if (d < a.dim) {
      v = __bfloat162float(x[d]);
      if (d < half) v = v * cs[d].x - __bfloat162float(x[d + half]) * cs[d].y;
      else if (d < a.rot) v = v * cs[d - half].x + __bfloat162float(x[d - half]) * cs[d - half].y;
    }
    out[e] = v * f;
  }
}

// ---- q, k, v of up to 128 tokens into shared memory ------------------------------------------------
struct RtHead {  // where a CTA's sequence and head lie
  const __nv_bfloat16* in;  // row 0 of the sequence
  int h, e0, ne, pos0;      // value columns [e0, e0 + ne)
};

// dst = src (16 bytes), or zeros
__device__ __forceinline__ void rt_cp16(uint32_t dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void rt_sync_workers() { asm volatile("barrier.sync 1, 512;" ::: "memory"); }
__device__ __forceinline__ void rt_cp_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// v of tokens t0 .. t0 + n - 1, asynchronously; zeros behind them and in the padding columns
template <int NV>
__device__ __forceinline__ void rt_load_v(const RetentionArgs& a, const RtHead& hd, int t0, int n, uint32_t sV, int tid) {
  constexpr int kStep = kRtWorkers / (8 * NV);  // rows from one of a thread's pieces to the next, a multiple of 8
  const int r0 = tid / (8 * NV), c = (tid % (8 * NV)) * 8;
  const bool col_ok = c < hd.ne;
  const __nv_bfloat16* src = hd.in + (long long)t0 * a.in_rs + a.v_col + hd.h * a.vdim + hd.e0 + (col_ok ? c : 0);  // a valid address for zeros too
  uint32_t dst = sV + (c >> 6) * kRtBlock + r0 * 128 + ((((c & 63) >> 3) ^ (r0 & 7)) << 4);
#pragma unroll
  for (int i = 0; i < 128 / kStep; ++i, dst += kStep * 128) {
    const int r = r0 + i * kStep;
    const bool live = col_ok && r < n;
    rt_cp16(dst, live ? src + (long long)r * a.in_rs : src, live);
  }
}

// k and v (and q and the gate) of n tokens to L2, a line at a time
template <bool ALL, int ND, int NV>
__device__ __forceinline__ void rt_prefetch(const RetentionArgs& a, const RtHead& hd, int t0, int n, int tid) {
  constexpr int kLines = (ALL ? 2 : 1) * (ND + NV);
  for (int it = tid; it < n * kLines; it += kRtWorkers) {
    const int r = it / kLines, x = it % kLines;
    const int col = x < ND ? a.k_col + hd.h * a.dim + min(x * 64, a.dim - 8) :
                    x < ND + NV ? a.v_col + hd.h * a.vdim + hd.e0 + min((x - ND) * 64, hd.ne - 8) :
                    x < 2 * ND + NV ? a.q_col + hd.h * a.dim + min((x - ND - NV) * 64, a.dim - 8) :
                                      a.g_col + hd.h * a.vdim + hd.e0 + min((x - 2 * ND - NV) * 64, hd.ne - 8);
    asm volatile("prefetch.global.L2 [%0];" ::"l"(hd.in + (long long)(t0 + r) * a.in_rs + col));
  }
}

// One pair of groups of eight columns (c, c + half) of a rotated vector times f.
__device__ __forceinline__ void rt_rotate_pair(uint8_t* dst, uint32_t lo_off, int r, int c, int half, const uint4& raw_u, const uint4& raw_v,
                                               const float* cx, const float* sx, float f) {
  const uint32_t wu[4] = {raw_u.x, raw_u.y, raw_u.z, raw_u.w}, wv[4] = {raw_v.x, raw_v.y, raw_v.z, raw_v.w};
  const uint64_t f2 = pack2(f, f), zero = 0ull;
  uint32_t xh[4], xl[4], yh[4], yl[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const uint64_t u = fma2(pack2(__uint_as_float(wu[i] << 16), __uint_as_float(wu[i] & 0xffff0000u)), f2, zero);
    const uint64_t v = fma2(pack2(__uint_as_float(wv[i] << 16), __uint_as_float(wv[i] & 0xffff0000u)), f2, zero);
    const uint64_t cc = pack2(cx[2 * i], cx[2 * i + 1]), ss = pack2(sx[2 * i], sx[2 * i + 1]), ns = pack2(-sx[2 * i], -sx[2 * i + 1]);
    rt_split2(fma2(u, cc, fma2(v, ns, zero)), xh[i], xl[i]);
    rt_split2(fma2(v, cc, fma2(u, ss, zero)), yh[i], yl[i]);
  }
  auto put = [&](int col, const uint32_t* hi, const uint32_t* lo) {
    uint8_t* p = dst + (col >> 6) * kRtBlock + r * 128 + ((((col & 63) >> 3) ^ (r & 7)) << 4);
    *reinterpret_cast<uint4*>(p) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(p + lo_off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  };
  put(c, xh, xl);
  put(c + half, yh, yl);
}

// q and k of up to 128 tokens where every dimension is rotated and dim = 64 ND.  A thread's items are pairs of groups of eight
// columns, kStep rows apart.  decay^(last - r) goes into row r of k, decay^(r + 1) into row r of q; `pw` holds the powers of
// the decay up to 128 (and beyond them they are formed here).
template <bool WITH_Q, int ND>
struct RtRows {
  static constexpr int kPairs = 4 * ND, kItems = 128 * kPairs / kRtWorkers, kStep = kRtWorkers / kPairs;
  uint4 k0[kItems], k1[kItems], q0[WITH_Q ? kItems : 1], q1[WITH_Q ? kItems : 1];

  __device__ __forceinline__ void load(const RetentionArgs& a, const RtHead& hd, int t0, int n, int tid) {
    const int r0 = tid / kPairs;
    const __nv_bfloat16* row = hd.in + (long long)(t0 + r0) * a.in_rs + hd.h * (64 * ND) + (tid % kPairs) * 8;
    const long long step = (long long)kStep * a.in_rs;
#pragma unroll
    for (int i = 0; i < kItems; ++i, row += step) {
      k0[i] = k1[i] = make_uint4(0u, 0u, 0u, 0u);
      if (WITH_Q) q0[i] = q1[i] = make_uint4(0u, 0u, 0u, 0u);
      if (r0 + i * kStep < n) {
        k0[i] = __ldg(reinterpret_cast<const uint4*>(row + a.k_col));
        k1[i] = __ldg(reinterpret_cast<const uint4*>(row + a.k_col + 32 * ND));
        if (WITH_Q) {
          q0[i] = __ldg(reinterpret_cast<const uint4*>(row + a.q_col));
          q1[i] = __ldg(reinterpret_cast<const uint4*>(row + a.q_col + 32 * ND));
        }
      }
    }
  }
  __device__ __forceinline__ void store(const RetentionArgs& a, const RtHead& hd, int t0, int n, int last, float l2, const float* pw, uint8_t* sK,
                                        uint8_t* sQ, uint32_t lo_off, int tid) const {
    const int r0 = tid / kPairs, c = (tid % kPairs) * 8, pos = hd.pos0 + t0;
    const bool ok = pos >= 0 && pos + n <= a.table_len;
    if (!ok && a.status) *a.status = 1;
    const float4* cs = reinterpret_cast<const float4*>(a.table + (long long)(pos + r0) * (32 * ND) + c);
#pragma unroll
    for (int i = 0; i < kItems; ++i, cs += kStep * 16 * ND) {
      const int r = r0 + i * kStep;
      float cx[8], sx[8];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float4 w = ok && r < n ? __ldg(cs + x) : make_float4(0.f, 0.f, 0.f, 0.f);
        cx[2 * x] = w.x; sx[2 * x] = w.y; cx[2 * x + 1] = w.z; sx[2 * x + 1] = w.w;
      }
      const int back = max(0, last - r);
      rt_rotate_pair(sK, lo_off, r, c, 32 * ND, k0[i], k1[i], cx, sx, (back <= 128 ? pw[back] : rt_pow(l2, back)) * a.k_scale);
      if (WITH_Q) rt_rotate_pair(sQ, lo_off, r, c, 32 * ND, q0[i], q1[i], cx, sx, pw[r + 1]);
    }
  }
};

// The same for any sizes, straight from global memory.
template <bool WITH_Q>
__device__ __forceinline__ void rt_build_any(const RetentionArgs& a, const RtHead& hd, int t0, int n, int last, float l2, uint8_t* sK, uint8_t* sQ,
                                             int nd, int tid) {
  const int half = a.rot >> 1;
  const bool wide = half % 8 == 0;
  const uint32_t lo_off = nd * kRtBlock;
  const int gr = wide ? half / 8 : 0;               // pairs of rotated groups of 8 per row
  const int gp = nd * 8 - (wide ? a.rot / 8 : 0);   // groups handled one by one (passed, padding, or all)
  const int per_row = gr + gp;
  for (int it = tid; it < 128 * per_row; it += kRtWorkers) {
    const int r = it / per_row, g = it - r * per_row;
    const bool live = r < n;
    const int pos = hd.pos0 + t0 + r;
    const bool ok = pos >= 0 && pos < a.table_len;
    if (live && !ok && a.status) *a.status = 1;
    const float fq = rt_pow(l2, r + 1), fk = rt_pow(l2, max(0, last - r)) * a.k_scale;
    const __nv_bfloat16* row = hd.in + (long long)(t0 + (live ? r : 0)) * a.in_rs + hd.h * a.dim;
    const __nv_bfloat16 *xq = row + a.q_col, *xk = row + a.k_col;
    const float2* cs = a.table + (long long)(ok ? pos : 0) * half;
    if (g < gr) {
      const int c = g * 8;
      float cx[8], sx[8];
#pragma unroll
      for (int i = 0; i < 8; i += 2) {
        const float4 t = *reinterpret_cast<const float4*>(cs + c + i);
        cx[i] = t.x; sx[i] = t.y; cx[i + 1] = t.z; sx[i + 1] = t.w;
      }
      const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
      rt_rotate_pair(sK, lo_off, r, c, half, live ? *reinterpret_cast<const uint4*>(xk + c) : zero,
                     live ? *reinterpret_cast<const uint4*>(xk + c + half) : zero, cx, sx, fk);
      if (WITH_Q)
        rt_rotate_pair(sQ, lo_off, r, c, half, live ? *reinterpret_cast<const uint4*>(xq + c) : zero,
                       live ? *reinterpret_cast<const uint4*>(xq + c + half) : zero, cx, sx, fq);
    } else {
      const int c = (wide ? a.rot : 0) + (g - gr) * 8;
      float x[8], y[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) x[i] = y[i] = 0.f;
      if (live) rt_group(a, wide, xk, cs, c, fk, x);
      rt_store8(sK, lo_off, r, c, x);
      if (WITH_Q) {
        if (live) rt_group(a, wide, xq, cs, c, fq, y);
        rt_store8(sQ, lo_off, r, c, y);
      }
    }
  }
}

__device__ __forceinline__ RtHead rt_head(const RtParams& p, int s, int h, int slice) {
  RtHead hd;
  hd.in = static_cast<const __nv_bfloat16*>(p.a.in) + (long long)s * p.a.Tn * p.a.in_rs;
  hd.h = h;
  hd.e0 = slice * 128;
  hd.ne = min(128, p.a.vdim - hd.e0);
  hd.pos0 = p.a.pos0[s] + (p.a.step_ptr ? *p.a.step_ptr : 0);
  return hd;
}

// ---- what each segment adds to the state: sum_j decay^(L-1-j) k_j v_j^T over its L tokens -----------------------
// Every k is brought into the frame of the segment's end, so the products of all tiles accumulate without a rescale (a factor
// too small for fp32 belongs to a token that no longer counts).  Two buffers: a tile is built while the one before is
// multiplied.
template <int ND, int NV, bool PLAIN>
__global__ void __launch_bounds__(kRtThreads, 1) retention_state_kernel(const RtParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const RetentionArgs& a = p.a;
  constexpr uint32_t lo_off = ND * kRtBlock, buf_bytes = (2 * ND + NV) * kRtBlock;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + 2 * buf_bytes + (ND < 2 ? kRtBlock : 0));  // a key of one block is read as a pair
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* pw = reinterpret_cast<float*>(bars + 8);  // [129] powers of the decay
  const uint32_t bar = smem_u32(bars);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

  int id = blockIdx.x;
  const int seg = id % (p.n_seg - 1);
  id /= p.n_seg - 1;
  const int slice = id % p.n_slice;
  id /= p.n_slice;
  const int h = id % a.H, s = id / a.H;
  const RtHead hd = rt_head(p, s, h, slice);
  const int t_begin = seg * p.seg_len, t_end = min(a.Tn, t_begin + p.seg_len);
  const float l2 = log2f(a.decay[h]);
  if (tid <= 128) pw[tid] = rt_pow(l2, tid);

  if (tid == 0) {
    *abort_flag = 0;
    mbar_init(bar, 1);
    mbar_init(bar + 8, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    fence_async_smem();
  }
  if (warp == 0) {
    tmem_alloc(smem_u32(tmem_slot), 128);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint64_t dM = smem_desc(0, kRtBlock, 1024);
  constexpr uint32_t idesc_s = instr_desc(64 * NV, true) | (1u << 15);

  bool fail = false;
  int tile = 0;
  RtRows<false, ND> next;
  // v of a tile comes by cp.async while the tile before is finished, k through registers
  auto fetch = [&](int t0, int b) {
    const int n = min(kRtChunk, t_end - t0);
    rt_load_v<NV>(a, hd, t0, n, smem_u32(smem + b * buf_bytes + 2 * ND * kRtBlock), tid);
    if (PLAIN) next.load(a, hd, t0, n, tid);
    rt_prefetch<false, ND, NV>(a, hd, t0 + kRtChunk, max(0, min(kRtChunk, t_end - t0 - kRtChunk)), tid);
  };
  if (warp < 16) fetch(t_begin, 0);
  for (int t0 = t_begin; t0 < t_end; t0 += kRtChunk, ++tile) {
    const int n = min(kRtChunk, t_end - t0), b = tile & 1;
    uint8_t* sK = smem + b * buf_bytes;
    if (warp < 16) {
      if (PLAIN) next.store(a, hd, t0, n, t_end - 1 - t0, l2, pw, sK, nullptr, lo_off, tid);
      else rt_build_any<false>(a, hd, t0, n, t_end - 1 - t0, l2, sK, nullptr, ND, tid);
      rt_cp_wait();
      fence_async_smem();
    }
    if (__syncthreads_or(fail ? 1 : 0)) {
      fail = true;
      break;
    }
    if (warp == 16 && lane == 0) {
      tc_fence_after();
      const uint32_t aK = smem_u32(sK), aV = aK + 2 * ND * kRtBlock;
      umma_ss8<128, 512, 128, 512>(tmem, dM + (aK >> 4), dM + (aV >> 4), idesc_s, tile > 0 ? 1u : 0u);
      umma_ss8<128, 512, 128, 512>(tmem, dM + ((aK + lo_off) >> 4), dM + (aV >> 4), idesc_s, 1u);
      umma_commit(bar + 8 * b);
    }
    if (warp < 16 && t0 + kRtChunk < t_end) {
      if (tile >= 1 && !wait_or_abort(bar + 8 * (b ^ 1), ((tile - 1) >> 1) & 1u, abort_flag, 63)) fail = true;  // the other buffer has been read
      fetch(t0 + kRtChunk, b ^ 1);
    }
  }
  rt_cp_wait();
  // the last two tiles' products (the others were waited for)
  for (int t = max(0, tile - 2); t < tile; ++t)
    if (!wait_or_abort(bar + 8 * (t & 1), (t >> 1) & 1u, abort_flag, 64)) fail = true;
  fail = __any_sync(0xffffffffu, fail);
  tc_fence_after();
  if (warp < 16 && !fail) {
    const int row = (warp & 3) * 32 + lane;
    float* dst = p.seg_state + (((long long)s * a.H + h) * (p.n_seg - 1) + seg) * a.dim * a.vdim + hd.e0 + (long long)row * a.vdim;
    for (int c = warp >> 2; c < 2 * NV; c += 4) {
      float v[32];
      tmem_ld32(tmem + ((uint32_t)((warp & 3) * 32) << 16) + c * 32, v);
      if (row < a.dim) {
#pragma unroll
        for (int i = 0; i < 32; i += 4)
          if (c * 32 + i < hd.ne) *reinterpret_cast<float4*>(dst + c * 32 + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
      }
    }
  }
  if (fail && lane == 0 && a.status) atomicExch(a.status, *abort_flag ? *abort_flag : 63);
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, 128);
}

// ---- from what each segment adds to the state behind each segment, in place ---------------------------------------
// Thread per four numbers of a head's state; carried in: a.state_in (or zeros).
__global__ void __launch_bounds__(256) retention_prefix_kernel(const RtParams p, long long per_head4) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= per_head4) return;
  const int sh = blockIdx.y;  // sequence * H + head
  const float f = rt_pow(log2f(p.a.decay[sh % p.a.H]), p.seg_len);
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  if (p.a.state_in) acc = reinterpret_cast<const float4*>(p.a.state_in)[sh * per_head4 + i];
  float4* seg = reinterpret_cast<float4*>(p.seg_state) + (long long)sh * (p.n_seg - 1) * per_head4 + i;
  const int n = p.n_seg - 1;  // every segment but the last is full
  for (int r0 = 0; r0 < n; r0 += 8) {
    float4 u[8];
#pragma unroll
    for (int r = 0; r < 8; ++r)
      if (r0 + r < n) u[r] = seg[(r0 + r) * per_head4];
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      if (r0 + r < n) {
        acc = make_float4(fmaf(f, acc.x, u[r].x), fmaf(f, acc.y, u[r].y), fmaf(f, acc.z, u[r].z), fmaf(f, acc.w, u[r].w));
        seg[(r0 + r) * per_head4] = acc;
      }
    }
  }
}

// ---- the chunks -----------------------------------------------------------------------------------
template <int ND, int NV, bool PLAIN>
__global__ void __launch_bounds__(kRtThreads, 1) retention_tc_kernel(const RtParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const RetentionArgs& a = p.a;
  constexpr int dimp = ND * 64;
  constexpr uint32_t q_lo = ND * kRtBlock;   // distance from a high term to its low term
  constexpr uint32_t s_lo = NV * kRtBlock;
  uint8_t* sK = smem;
  uint8_t* sV = sK + 2 * ND * kRtBlock;
  uint8_t* sQ = sV + NV * kRtBlock;
  uint8_t* sS = sQ + 2 * ND * kRtBlock;
  // o on its way to memory takes the place of q^ and part of the state's; row sums of squares [2 NV][128] the end of the latter
  float* ssq = reinterpret_cast<float*>(sS + 2 * NV * kRtBlock) - 2 * NV * 128;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sS + 2 * NV * kRtBlock);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 4);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* pw = reinterpret_cast<float*>(bars + 8);  // [129] powers of the decay
  const uint32_t bar_a = smem_u32(bars), bar_o = bar_a + 8, bar_s = bar_a + 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

  int id = blockIdx.x;
  const int seg = id % p.n_seg;
  id /= p.n_seg;
  const int slice = id % p.n_slice;
  id /= p.n_slice;
  const int h = id % a.H, s = id / a.H;
  const RtHead hd = rt_head(p, s, h, slice);
  const int e0 = hd.e0, ne = hd.ne;
  const int t_begin = seg * p.seg_len, t_end = min(a.Tn, t_begin + p.seg_len);
  const float l2 = log2f(a.decay[h]);
  if (tid <= 128) pw[tid] = rt_pow(l2, tid);

  if (tid == 0) {
    *abort_flag = 0;
    for (int i = 0; i < 3; ++i) mbar_init(bar_a + 8 * i, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    fence_async_smem();
  }
  if (warp == 0) {
    tmem_alloc(smem_u32(tmem_slot), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const int chunk = max(1, min(kRtChunk, l2 < 0.f ? (int)(40.f / -l2) : kRtChunk));
  unsigned done = 0;  // chunks finished

  if (warp == 16) {
    // ================= MMA issuer =================
    const uint64_t dK = smem_desc(0, 16, 1024), dM = smem_desc(0, kRtBlock, 1024);  // K-major rows; MN-major blocks
    constexpr uint32_t kIdescA = instr_desc(128, false), idesc_o = instr_desc(64 * NV, true), idesc_s = idesc_o | (1u << 15);  // 15: A read MN-major
    const uint32_t aK = smem_u32(sK), aV = smem_u32(sV), aQ = smem_u32(sQ), aS = smem_u32(sS);
    for (int t0 = t_begin; t0 < t_end; ++done) {
      t0 += min(chunk, t_end - t0);
      if (__syncthreads_or(0)) break;  // the operands are there
      if (lane == 0) {
        tc_fence_after();
        // A = q^ k^T: high x high, high x low, low x high
#pragma unroll 1
        for (int t = 0; t < 3; ++t) {
          const uint64_t da = dK + ((aQ + (t == 2 ? q_lo : 0)) >> 4), db = dK + ((aK + (t == 1 ? q_lo : 0)) >> 4);
          if constexpr (ND == 2) umma_ss8<2, kRtBlock / 16, 2, kRtBlock / 16>(tmem + kRtA, da, db, kIdescA, t);
          else umma_ss4<2, 2>(tmem + kRtA, da, db, kIdescA, t);
        }
        umma_commit(bar_a);
        // o = q^ S
#pragma unroll 1
        for (int t = 0; t < 3; ++t) {
          const uint64_t da = dK + ((aQ + (t == 2 ? q_lo : 0)) >> 4), db = dM + ((aS + (t == 1 ? s_lo : 0)) >> 4);
          if constexpr (ND == 2) umma_ss8<2, kRtBlock / 16, 128, 512>(tmem + kRtO, da, db, idesc_o, t);
          else umma_ss4<2, 128>(tmem + kRtO, da, db, idesc_o, t);
        }
      }
      __syncwarp();
      if (__syncthreads_or(0)) {  // P is there, and the state has been scaled
        if (lane == 0) umma_commit(bar_o);  // completes with the products above
        break;
      }
      if (lane == 0) {
        tc_fence_after();
        // o += P v
        umma_ts_chain<8>(tmem + kRtO, tmem + kRtPh, dM + (aV >> 4), idesc_o, 1u);
        umma_ts_chain<8>(tmem + kRtO, tmem + kRtPl, dM + (aV >> 4), idesc_o, 1u);
        umma_commit(bar_o);
        // S += k^^T v
        umma_ss8<128, 512, 128, 512>(tmem + kRtS, dM + (aK >> 4), dM + (aV >> 4), idesc_s, 1u);
        umma_ss8<128, 512, 128, 512>(tmem + kRtS, dM + ((aK + q_lo) >> 4), dM + (aV >> 4), idesc_s, 1u);
        umma_commit(bar_s);
      }
      __syncwarp();
    }
  } else {
    // ================= everything else: four threads per row, a part of its columns each =================
    const int quarter = warp & 3, part = warp >> 2, row = quarter * 32 + lane;
    const uint32_t lane_addr = tmem + ((uint32_t)(quarter * 32) << 16);
    const int c = part;              // this thread's 32-column piece of o and of the state,
    const bool has_piece = c < 2 * NV;  // if there are that many
    const long long st0 = ((long long)s * a.H + h) * a.dim * a.vdim + e0;                  // this head's slice of the carried state
    const long long sg0 = ((long long)s * a.H + h) * (p.n_seg - 1) * a.dim * a.vdim + e0;  // and of the segments' states
    rt_load_v<NV>(a, hd, t_begin, min(chunk, t_end - t_begin), smem_u32(sV), tid);

    // state columns [32 c + 16 q, +16) of this thread's key dimension into shared memory, the B operand of the next chunk
    auto share_state = [&](int q, const float* v) {
      if (row < dimp) {
        rt_store8(sS, s_lo, row, c * 32 + q * 16, v);
        rt_store8(sS, s_lo, row, c * 32 + q * 16 + 8, v + 8);
      }
    };
    // ---- the state in front of the segment ----
    if (has_piece) {
      float v[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) v[i] = 0.f;
      if (row < a.dim) {
        const float* src = seg > 0 ? p.seg_state + sg0 + (long long)(seg - 1) * a.dim * a.vdim : a.state_in ? a.state_in + st0 : nullptr;
        if (src) {
          src += (long long)row * a.vdim + c * 32;
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            if (c * 32 + i < ne) {  // ne is a multiple of 8
              const float4 t = *reinterpret_cast<const float4*>(src + i);
              v[i] = t.x; v[i + 1] = t.y; v[i + 2] = t.z; v[i + 3] = t.w;
            }
          }
        }
      }
      tmem_st32(lane_addr + kRtS + c * 32, v);
      share_state(0, v);
      share_state(1, v + 16);
    }
    tc_wait_st();

    bool fail = false;
    for (int t0 = t_begin; t0 < t_end; ++done) {
      const int n = min(chunk, t_end - t0), t1 = t0 + n, n1 = min(chunk, t_end - t1);
      const uint32_t par = done & 1u;
      if (PLAIN) {
        RtRows<true, ND> qk;
        qk.load(a, hd, t0, n, tid);
        qk.store(a, hd, t0, n, n - 1, l2, pw, sK, sQ, q_lo, tid);
      } else rt_build_any<true>(a, hd, t0, n, n - 1, l2, sK, sQ, ND, tid);
      rt_cp_wait();
      fence_async_smem();
      tc_fence_before();
      if (__syncthreads_or(fail ? 1 : 0)) {
        fail = true;
        break;
      }
      tc_fence_after();
      rt_prefetch<true, ND, NV>(a, hd, t1, n1, tid);  // the next chunk's rows come to L2 while this one is worked on
      // ---- state *= decay^n, while the scores are formed ----
      {
        const float f = pw[n];
        if (has_piece) {
          float v[32];
          tmem_ld32(lane_addr + kRtS + c * 32, v);
#pragma unroll
          for (int i = 0; i < 32; ++i) v[i] *= f;
          tmem_st32(lane_addr + kRtS + c * 32, v);
        }
      }
      // ---- P ----
      if (!wait_or_abort(bar_a, par, abort_flag, 60)) fail = true;
      fail = __any_sync(0xffffffffu, fail);  // the loads below are collective
      tc_fence_after();
      {
        const float f = rt_pow(-l2, n);
        uint32_t hi[16], lo[16];
        if (part > quarter) {  // keys behind every query of this warp
#pragma unroll
          for (int i = 0; i < 16; ++i) hi[i] = lo[i] = 0u;
        } else {
          float v[32];
          tmem_ld32(lane_addr + kRtA + part * 32, v);
          if (part == quarter) {
#pragma unroll
            for (int i = 0; i < 32; ++i) v[i] = i <= lane ? v[i] : 0.f;
          }
          const uint64_t f2 = pack2(f, f);
#pragma unroll
          for (int i = 0; i < 16; ++i) rt_split2(fma2(pack2(v[2 * i], v[2 * i + 1]), f2, 0ull), hi[i], lo[i]);
        }
        tmem_st16(lane_addr + kRtPh + part * 16, hi);
        tmem_st16(lane_addr + kRtPl + part * 16, lo);
      }
      tc_wait_st();
      tc_fence_before();
      if (__syncthreads_or(fail ? 1 : 0)) {
        fail = true;
        break;
      }
      // the pieces of eight columns that this thread finishes: column 8 c8 of rows r0 + i kOutStep
      constexpr int kOutStep = kRtWorkers / (8 * NV);
      const int r0 = tid / (8 * NV), c8 = tid % (8 * NV);
      const bool col_ok = c8 * 8 < ne;
      const long long tok0 = (long long)s * a.Tn + t0 + r0;
      uint4 gate[2 * NV];  // on its way while the products run
      if (p.n_slice == 1) {
        const __nv_bfloat16* gp = hd.in + (long long)(t0 + r0) * a.in_rs + a.g_col + h * a.vdim + c8 * 8;
#pragma unroll
        for (int i = 0; i < 2 * NV; ++i, gp += (long long)kOutStep * a.in_rs) {
          gate[i] = make_uint4(0u, 0u, 0u, 0u);
          if (col_ok && r0 + i * kOutStep < n) gate[i] = __ldg(reinterpret_cast<const uint4*>(gp));
        }
      }
      // ---- o: head norm, gate, store; rows go through shared memory (q^ and the old state have been read by then), so that
      // global accesses run along rows ----
      if (!wait_or_abort(bar_o, par, abort_flag, 61)) fail = true;
      fail = __any_sync(0xffffffffu, fail);
      tc_fence_after();
      {
        constexpr int kRowChunks = 16 * NV;  // 16-byte pieces of a row of o, swizzled by the row
        float4* so = reinterpret_cast<float4*>(sQ);
        if (has_piece) {
          float v[32], ss = 0.f;
          tmem_ld32(lane_addr + kRtO + c * 32, v);
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            ss += (v[4 * i] * v[4 * i] + v[4 * i + 1] * v[4 * i + 1]) + (v[4 * i + 2] * v[4 * i + 2] + v[4 * i + 3] * v[4 * i + 3]);
            so[row * kRowChunks + ((c * 8 + i) ^ (row & 7))] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
          }
          ssq[c * 128 + row] = ss;  // padding columns hold zeros
        }
        rt_sync_workers();
        const float inv_ne = 1.f / (float)ne;
        __nv_bfloat16* yp = static_cast<__nv_bfloat16*>(a.y) + tok0 * a.y_rs + h * a.vdim + c8 * 8;
#pragma unroll
        for (int i = 0; i < 2 * NV; ++i, yp += (long long)kOutStep * a.y_rs) {
          const int r = r0 + i * kOutStep;
          if (col_ok && r < n) {
            const float4 x = so[r * kRowChunks + ((2 * c8) ^ (r & 7))], y = so[r * kRowChunks + ((2 * c8 + 1) ^ (r & 7))];
            if (p.n_slice > 1) {  // the norm needs the other slices too: o as it is, for head_norm_gate_kernel
              float4* dst = reinterpret_cast<float4*>(a.o + ((tok0 + i * kOutStep) * a.H + h) * a.vdim + e0 + c8 * 8);
              dst[0] = x;
              dst[1] = y;
            } else {
              float ss = 0.f;
#pragma unroll
              for (int k = 0; k < 2 * NV; ++k) ss += ssq[k * 128 + r];
              const float inv = rsqrtf(fmaf(ss, inv_ne, a.eps));
              float v[8] = {x.x, x.y, x.z, x.w, y.x, y.y, y.z, y.w}, g[8];
              unpack16<__nv_bfloat16>(gate[i], g);
#pragma unroll
              for (int k = 0; k < 8; ++k) v[k] *= __fdividef(g[k], 1.f + __expf(-g[k]));
              st16<__nv_bfloat16>(yp, v, inv);
            }
          }
        }
        rt_sync_workers();
      }
      // ---- the state behind the chunk ----
      if (!wait_or_abort(bar_s, par, abort_flag, 62)) fail = true;
      fail = __any_sync(0xffffffffu, fail);
      tc_fence_after();
      if (n1 > 0) rt_load_v<NV>(a, hd, t1, n1, smem_u32(sV), tid);
      if (n1 > 0 || (t_end == a.Tn && a.state_out)) {
        if (has_piece) {
#pragma unroll
          for (int q = 0; q < 2; ++q) {  // 16 columns at a time: the fetched rows hold many registers
            float v[16];
            tmem_ld16_nowait(lane_addr + kRtS + c * 32 + q * 16, v);
            tc_wait_ld();
            if (n1 > 0) {
              share_state(q, v);
            } else if (row < a.dim && !fail) {
              float* dst = a.state_out + st0 + (long long)row * a.vdim + c * 32 + q * 16;
#pragma unroll
              for (int i = 0; i < 16; i += 4)
                if (c * 32 + q * 16 + i < ne) *reinterpret_cast<float4*>(dst + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
            }
          }
        }
      }
      t0 = t1;
    }
    rt_cp_wait();
    if (fail && tid == 0 && a.status) atomicExch(a.status, *abort_flag ? *abort_flag : 60);
  }
  tc_fence_before();
  if (__syncthreads_or(*abort_flag) && tid == 0) {  // give what may be in flight a bounded chance to finish
    const uint32_t par = done & 1u;
    mbar_wait(bar_a, par, kRtDrainCycles);
    mbar_wait(bar_o, par, kRtDrainCycles);
    mbar_wait(bar_s, par, kRtDrainCycles);
  }
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, 512);
}

static size_t rt_smem_main(int nd, int nv) {
  const size_t bytes = (size_t)(4 * nd + 3 * nv) * kRtBlock + 64 + 520 + 1024;
  return bytes < 120 * 1024 ? 120 * 1024 : bytes;  // one CTA owns an SM (it allocates all of TMEM)
}
static size_t rt_smem_state(int nd, int nv) { return (size_t)(2 * (2 * nd + nv) + (nd < 2 ? 1 : 0)) * kRtBlock + 64 + 520 + 1024; }

template <int ND, int NV, bool PLAIN>
static int rt_launch(const RtParams& p, cudaStream_t st) {
  static bool ready[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) {
    set_error("retention: cudaGetDevice failed");
    return DGPT_E_CUDA;
  }
  if (!ready[dev]) {
    cudaError_t e = cudaFuncSetAttribute(retention_state_kernel<ND, NV, PLAIN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)rt_smem_state(ND, NV));
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(retention_tc_kernel<ND, NV, PLAIN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)rt_smem_main(ND, NV));
    if (e != cudaSuccess) {
      set_error("retention: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
      return DGPT_E_CUDA;
    }
    ready[dev] = true;
  }
  const int heads = p.a.n_seq * p.a.H * p.n_slice;
  if (p.n_seg > 1) {
    retention_state_kernel<ND, NV, PLAIN><<<heads * (p.n_seg - 1), kRtThreads, rt_smem_state(ND, NV), st>>>(p);
    if (int e = launch_status("retention_state")) return e;
    const long long per_head4 = (long long)p.a.dim * p.a.vdim / 4;
    retention_prefix_kernel<<<dim3((unsigned)((per_head4 + 255) / 256), (unsigned)(p.a.n_seq * p.a.H)), 256, 0, st>>>(p, per_head4);
    if (int e = launch_status("retention_prefix")) return e;
  }
  retention_tc_kernel<ND, NV, PLAIN><<<heads * p.n_seg, kRtThreads, rt_smem_main(ND, NV), st>>>(p);
  return launch_status("retention_tc");
}

}  // namespace tc

static int rt_segments(int n_seq, int H, int n_slice, int T) {
  const int want = 148 / (n_seq * H * n_slice);  // CTAs of one wave
  const int most = (T + 255) / 256;
  return want < 1 ? 1 : (want < most ? want : most);
}
size_t retention_tc_workspace_bytes(int n_seq, int T, int H, int dim, int vdim) {
  const int n_seg = rt_segments(n_seq, H, (vdim + 127) / 128, T);
  return (size_t)n_seq * H * (n_seg - 1) * dim * vdim * sizeof(float);
}

bool retention_tc_supported(const RetentionArgs& a, int dtype, float min_decay) {
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  if (dtype != DGPT_BF16 || a.dim > 128 || a.dim % 8 || a.vdim % 8 || a.in_rs % 8 || a.y_rs % 8) return false;
  if (a.q_col % 8 || a.k_col % 8 || a.v_col % 8 || a.g_col % 8 || !al16(a.in) || !al16(a.y) || !al16(a.table)) return false;
  if ((a.state_in && !al16(a.state_in)) || (a.state_out && !al16(a.state_out))) return false;
  if (!(min_decay >= 0.0625f)) return false;  // chunks of ten tokens and less: the recurrent form
  return tc::device_is_sm100();
}

int retention_tc_launch(const RetentionArgs& a, float* seg_state, cudaStream_t st) {
  using namespace tc;
  RtParams p;
  p.a = a;
  p.n_slice = (a.vdim + 127) / 128;
  p.n_seg = rt_segments(a.n_seq, a.H, p.n_slice, a.Tn);
  p.seg_len = ((a.Tn + p.n_seg - 1) / p.n_seg + kRtChunk - 1) / kRtChunk * kRtChunk;
  p.n_seg = (a.Tn + p.seg_len - 1) / p.seg_len;
  const int nd = (a.dim + 63) / 64, nv = a.vdim > 64 ? 2 : 1;  // 64-column blocks of a key and of a value slice
  p.seg_state = seg_state;
  const bool plain = a.rot == a.dim && a.dim == 64 * nd;  // every dimension rotated, no padding
#define DGPT_RT(ND, NV) return plain ? rt_launch<ND, NV, true>(p, st) : rt_launch<ND, NV, false>(p, st)
  if (nd == 1 && nv == 1) DGPT_RT(1, 1);
  if (nd == 1) DGPT_RT(1, 2);
  if (nv == 1) DGPT_RT(2, 1);
  DGPT_RT(2, 2);
#undef DGPT_RT
}

}  // namespace dgpt
