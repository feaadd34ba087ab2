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
// One CTA of 256 threads per (sequence, head, 128 value columns, segment of the tokens).  Few heads leave most SMs idle, so
// a long sequence is cut into segments: a first launch (STATE_ONLY) forms each segment's own contribution to the state,
// the second starts each segment from the decayed sum of those before it.
//   all threads     rotate, split and write q^, k^, v of a chunk into swizzled shared memory; A -> P; state -> shared memory;
//                   head norm, output gate and store
//   thread 0        issues the products
// TMEM columns: A [0, 128)  P high [128, 192)  P low [192, 256)  o [256, 384)  state [384, 512) (lane = key dimension).
// Every mbarrier wait is bounded; when one runs out the CTA leaves its loop together, waits (bounded) for what it issued,
// frees TMEM and reports through the status word.
#include "retention.cuh"
#include "tcgen05.cuh"

namespace dgpt {
namespace tc {

constexpr int kRtThreads = 256;
constexpr int kRtChunk = 128;
constexpr uint32_t kRtBlock = 128 * 128;  // [128 rows][64 columns] bf16, swizzled
constexpr uint32_t kRtA = 0, kRtPh = 128, kRtPl = 192, kRtO = 256, kRtS = 384;

struct RtParams {
  RetentionArgs a;
  int n_seg, seg_len, n_slice;
  int nd, nv;        // 64-column blocks of a key and of a value slice
  float* seg_state;  // [n_seq, H, n_seg - 1, dim, vdim]
};

__device__ __forceinline__ void rt_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
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

template <bool STATE_ONLY>
__global__ void __launch_bounds__(kRtThreads, 1) retention_tc_kernel(const RtParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const RetentionArgs& a = p.a;
  const int nd = p.nd, nv = p.nv, dimp = nd * 64;
  const uint32_t q_lo = nd * kRtBlock, s_lo = nv * kRtBlock;  // distance from a high term to its low term
  uint8_t* sK = smem;
  uint8_t* sV = sK + 2 * nd * kRtBlock;
  uint8_t* sQ = sV + nv * kRtBlock;
  uint8_t* sS = sQ + 2 * nd * kRtBlock;
  uint8_t* tail = STATE_ONLY ? sQ + (nd < 2 ? kRtBlock : 0) : sS + 2 * nv * kRtBlock;
  float* ssq = reinterpret_cast<float*>(tail);  // [2][128]
  uint64_t* bars = reinterpret_cast<uint64_t*>(ssq + 256);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 4);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const uint32_t bar_a = smem_u32(bars), bar_o = bar_a + 8, bar_s = bar_a + 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

  int id = blockIdx.x;
  const int n_seg_here = STATE_ONLY ? p.n_seg - 1 : p.n_seg;
  const int seg = id % n_seg_here;
  id /= n_seg_here;
  const int slice = id % p.n_slice;
  id /= p.n_slice;
  const int h = id % a.H, s = id / a.H;
  const int e0 = slice * 128, ne = min(128, a.vdim - e0);  // this CTA's value columns
  const int N = (ne + 15) / 16 * 16;
  const int t_begin = seg * p.seg_len, t_end = min(a.Tn, t_begin + p.seg_len);

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
  const int quarter = warp & 3, half_id = warp >> 2, row = quarter * 32 + lane;
  const uint32_t lane_addr = tmem + ((uint32_t)(quarter * 32) << 16);
  // 32-column pieces of o and of the state: the first half of them for one warp of a quarter, the rest for the other
  const int pieces = (N + 31) / 32, c_first = half_id == 0 ? 0 : (pieces + 1) / 2, c_last = half_id == 0 ? (pieces + 1) / 2 : pieces;

  const float decay = a.decay[h], l2 = log2f(decay);
  const int chunk = max(1, min(kRtChunk, l2 < 0.f ? (int)(40.f / -l2) : kRtChunk));
  const long long st0 = ((long long)s * a.H + h) * a.dim * a.vdim + e0;            // this head's slice of the carried state
  const long long sg0 = ((long long)s * a.H + h) * (p.n_seg - 1) * a.dim * a.vdim + e0;  // and of the segments' states
  const int pos0 = a.pos0[s] + (a.step_ptr ? *a.step_ptr : 0);

  // state columns [32 c, +32) of this thread's key dimension, TMEM -> shared memory as the B operand of the next chunk
  auto share_state = [&](int c, const float* v) {
    if (row < dimp) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (c * 32 + i * 8 < N) rt_store8(sS, s_lo, row, c * 32 + i * 8, v + i * 8);
    }
  };
  // ---- the state in front of the segment ----
  for (int c = c_first; c < c_last; ++c) {
    float v[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) v[i] = 0.f;
    if (!STATE_ONLY && row < a.dim) {
      for (int r = -1; r < seg; ++r) {  // -1: the state carried in
        if (r < 0 && a.state_in == nullptr) continue;
        const float f = rt_pow(l2, t_begin - (r + 1) * p.seg_len);
        const float* src = r < 0 ? a.state_in + st0 : p.seg_state + sg0 + (long long)r * a.dim * a.vdim;
        src += (long long)row * a.vdim + c * 32;
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          if (c * 32 + i < ne) {  // ne is a multiple of 8
            const float4 t = *reinterpret_cast<const float4*>(src + i);
            v[i] = fmaf(f, t.x, v[i]);
            v[i + 1] = fmaf(f, t.y, v[i + 1]);
            v[i + 2] = fmaf(f, t.z, v[i + 2]);
            v[i + 3] = fmaf(f, t.w, v[i + 3]);
          }
        }
      }
    }
    tmem_st32(lane_addr + kRtS + c * 32, v);
    if (!STATE_ONLY) share_state(c, v);
  }
  tc_wait_st();

  const uint64_t dK = smem_desc(0, 16, 1024), dM = smem_desc(0, kRtBlock, 1024);  // K-major rows; MN-major blocks
  const uint32_t kIdescA = instr_desc(128, false), idesc_o = instr_desc(N, true), idesc_s = idesc_o | (1u << 15);  // 15: A read MN-major
  const int half = a.rot >> 1;
  const bool wide_rot = half % 8 == 0;
  bool fail = false;
  unsigned done = 0;  // chunks finished
  int issued = 0;     // thread 0: products of the current chunk in flight (1: scores, 2: all)

  for (int t0 = t_begin; t0 < t_end; ++done) {
    const int n = min(chunk, t_end - t0);
    const uint32_t par = done & 1u;
    // ---- operands into shared memory ----
    {
      const int gr = wide_rot ? half / 8 : 0;                      // pairs of rotated groups of 8 per row
      const int gp = dimp / 8 - (wide_rot ? a.rot / 8 : 0);        // groups handled one by one (passed, padding, or all)
      const int per_row = gr + gp;
      for (int it = tid; it < 128 * per_row; it += kRtThreads) {
        const int r = it / per_row, g = it - r * per_row;
        const bool live = r < n;
        const int pos = pos0 + t0 + r;
        const bool ok = pos >= 0 && pos < a.table_len;
        if (live && !ok && a.status) *a.status = 1;
        const float fq = rt_pow(l2, r + 1), fk = live ? rt_pow(l2, n - 1 - r) * a.k_scale : 0.f;
        const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(a.in) + ((long long)s * a.Tn + t0 + (live ? r : 0)) * a.in_rs;
        const __nv_bfloat16 *xq = in + a.q_col + h * a.dim, *xk = in + a.k_col + h * a.dim;
        const float2* cs = a.table + (long long)(live && ok ? pos : 0) * half;
        if (g < gr) {
          const int c = g * 8;
          float cx[8], sx[8];
#pragma unroll
          for (int i = 0; i < 8; i += 2) {
            const float4 t = *reinterpret_cast<const float4*>(cs + c + i);
            cx[i] = t.x; sx[i] = t.y; cx[i + 1] = t.z; sx[i + 1] = t.w;
          }
          float u[8], v[8], x[8], y[8];
          ld16<__nv_bfloat16>(xk + c, u);
          ld16<__nv_bfloat16>(xk + c + half, v);
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            x[i] = live ? (u[i] * cx[i] - v[i] * sx[i]) * fk : 0.f;
            y[i] = live ? (v[i] * cx[i] + u[i] * sx[i]) * fk : 0.f;
          }
          rt_store8(sK, q_lo, r, c, x);
          rt_store8(sK, q_lo, r, c + half, y);
          if (!STATE_ONLY) {
            ld16<__nv_bfloat16>(xq + c, u);
            ld16<__nv_bfloat16>(xq + c + half, v);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              x[i] = live ? (u[i] * cx[i] - v[i] * sx[i]) * fq : 0.f;
              y[i] = live ? (v[i] * cx[i] + u[i] * sx[i]) * fq : 0.f;
            }
            rt_store8(sQ, q_lo, r, c, x);
            rt_store8(sQ, q_lo, r, c + half, y);
          }
        } else {
          const int c = (wide_rot ? a.rot : 0) + (g - gr) * 8;
          float x[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) x[i] = 0.f;
          if (live) rt_group(a, wide_rot, xk, cs, c, fk, x);
          rt_store8(sK, q_lo, r, c, x);
          if (!STATE_ONLY) {
#pragma unroll
            for (int i = 0; i < 8; ++i) x[i] = 0.f;
            if (live) rt_group(a, wide_rot, xq, cs, c, fq, x);
            rt_store8(sQ, q_lo, r, c, x);
          }
        }
      }
      const int gv = N / 8;
      for (int it = tid; it < 128 * gv; it += kRtThreads) {
        const int r = it / gv, c = (it - r * gv) * 8;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < n && c < ne)
          v = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.in) + ((long long)s * a.Tn + t0 + r) * a.in_rs + a.v_col +
                                              h * a.vdim + e0 + c);
        *reinterpret_cast<uint4*>(sV + (c >> 6) * kRtBlock + r * 128 + ((((c & 63) >> 3) ^ (r & 7)) << 4)) = v;
      }
    }
    fence_async_smem();
    tc_fence_before();
    __syncthreads();
    const uint32_t aK = smem_u32(sK), aV = smem_u32(sV), aQ = smem_u32(sQ), aS = smem_u32(sS);
    if (!STATE_ONLY && tid == 0) {
      tc_fence_after();
      const int steps = dimp / 16;
      // A = q^ k^T: high x high, high x low, low x high
      for (int t = 0; t < 3; ++t) {
        const uint32_t qa = aQ + (t == 2 ? q_lo : 0), ka = aK + (t == 1 ? q_lo : 0);
        for (int ks = 0; ks < steps; ++ks) {
          const uint32_t off = (uint32_t)(ks >> 2) * kRtBlock + (uint32_t)(ks & 3) * 32u;
          umma_ss(tmem + kRtA, dK + ((qa + off) >> 4), dK + ((ka + off) >> 4), kIdescA, t > 0 || ks > 0 ? 1u : 0u);
        }
      }
      umma_commit(bar_a);
      // o = q^ S
      for (int t = 0; t < 3; ++t) {
        const uint32_t qa = aQ + (t == 2 ? q_lo : 0), sa = aS + (t == 1 ? s_lo : 0);
        for (int ks = 0; ks < steps; ++ks) {
          const uint32_t off = (uint32_t)(ks >> 2) * kRtBlock + (uint32_t)(ks & 3) * 32u;
          umma_ss(tmem + kRtO, dK + ((qa + off) >> 4), dM + ((sa + ks * 2048) >> 4), idesc_o, t > 0 || ks > 0 ? 1u : 0u);
        }
      }
      issued = 1;
    }
    // ---- state *= decay^n, while the scores are formed ----
    tc_fence_after();
    {
      const float f = rt_pow(l2, n);
      for (int c = c_first; c < c_last; ++c) {
        float v[32];
        tmem_ld32(lane_addr + kRtS + c * 32, v);
#pragma unroll
        for (int i = 0; i < 32; ++i) v[i] *= f;
        tmem_st32(lane_addr + kRtS + c * 32, v);
      }
    }
    // ---- P ----
    if (!STATE_ONLY) {
      if (!wait_or_abort(bar_a, par, abort_flag, 60)) fail = true;
      fail = __any_sync(0xffffffffu, fail);  // the loads below are collective
      tc_fence_after();
      const float f = rt_pow(-l2, n);
      const int j0 = half_id * 64;
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        float v[32];
        tmem_ld32(lane_addr + kRtA + j0 + c * 32, v);
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int j = j0 + c * 32 + 2 * i;
          rt_split(j <= row ? v[2 * i] * f : 0.f, j + 1 <= row ? v[2 * i + 1] * f : 0.f, hi[i], lo[i]);
        }
        tmem_st16(lane_addr + kRtPh + (j0 >> 1) + c * 16, hi);
        tmem_st16(lane_addr + kRtPl + (j0 >> 1) + c * 16, lo);
      }
    }
    tc_wait_st();
    tc_fence_before();
    if (__syncthreads_or(fail ? 1 : 0)) {
      fail = true;
      break;
    }
    if (tid == 0) {
      tc_fence_after();
      if (!STATE_ONLY) {
        // o += P v
        for (int t = 0; t < 2; ++t)
          umma_ts_chain<8>(tmem + kRtO, tmem + (t == 0 ? kRtPh : kRtPl), dM + (aV >> 4), idesc_o, 1u);
        umma_commit(bar_o);
      }
      // S += k^^T v
      for (int t = 0; t < 2; ++t) {
        const uint32_t ka = aK + (t == 1 ? q_lo : 0);
        for (int ks = 0; ks < 8; ++ks) umma_ss(tmem + kRtS, dM + ((ka + ks * 2048) >> 4), dM + ((aV + ks * 2048) >> 4), idesc_s, 1u);
      }
      umma_commit(bar_s);
      issued = 2;
    }
    // ---- o: head norm, gate, store ----
    if (!STATE_ONLY) {
      if (!wait_or_abort(bar_o, par, abort_flag, 61)) fail = true;
      fail = __any_sync(0xffffffffu, fail);
      tc_fence_after();
      const bool live = row < n;
      const long long tok = (long long)s * a.Tn + t0 + row;
      float v[2][32];
      float ss = 0.f;
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        if (c_first + c < c_last) {
          tmem_ld32(lane_addr + kRtO + (c_first + c) * 32, v[c]);
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if ((c_first + c) * 32 + i < ne) ss += v[c][i] * v[c][i];
        }
      }
      if (p.n_slice > 1) {  // the norm needs the other slices too: o as it is, for head_norm_gate_kernel
#pragma unroll
        for (int c = 0; c < 2; ++c)
          if (c_first + c < c_last && live) {
            float* dst = a.o + (tok * a.H + h) * a.vdim + e0 + (c_first + c) * 32;
#pragma unroll
            for (int i = 0; i < 32; i += 4)
              if ((c_first + c) * 32 + i < ne) *reinterpret_cast<float4*>(dst + i) = make_float4(v[c][i], v[c][i + 1], v[c][i + 2], v[c][i + 3]);
          }
      } else {
        ssq[half_id * 128 + row] = ss;
        asm volatile("barrier.sync %0, 64;" ::"r"(1 + quarter) : "memory");  // the two warps of this quarter
        const float inv = rsqrtf((ssq[row] + ssq[128 + row]) / (float)ne + a.eps);
        const __nv_bfloat16* gp = static_cast<const __nv_bfloat16*>(a.in) + (live ? tok : 0) * a.in_rs + a.g_col + h * a.vdim;
        __nv_bfloat16* yp = static_cast<__nv_bfloat16*>(a.y) + tok * a.y_rs + h * a.vdim;
#pragma unroll
        for (int c = 0; c < 2; ++c)
          if (c_first + c < c_last && live) {
            const int col = (c_first + c) * 32;
#pragma unroll
            for (int i = 0; i < 32; i += 8)
              if (col + i < ne) {
                float gv[8];
                ld16<__nv_bfloat16>(gp + col + i, gv);
#pragma unroll
                for (int k = 0; k < 8; ++k) gv[k] = v[c][i + k] * __fdividef(gv[k], 1.f + __expf(-gv[k]));
                st16<__nv_bfloat16>(yp + col + i, gv, inv);
              }
          }
        asm volatile("barrier.sync %0, 64;" ::"r"(1 + quarter) : "memory");  // `ssq` may be written again
      }
    }
    // ---- the state behind the chunk ----
    if (!wait_or_abort(bar_s, par, abort_flag, 62)) fail = true;
    fail = __any_sync(0xffffffffu, fail);
    tc_fence_after();
    t0 += n;
    const bool last = t0 >= t_end;
    if (!STATE_ONLY || last) {
      for (int c = c_first; c < c_last; ++c) {
        float v[32];
        tmem_ld32(lane_addr + kRtS + c * 32, v);
        if (!last) {
          share_state(c, v);
        } else {
          float* dst = nullptr;
          if (STATE_ONLY) dst = p.seg_state + sg0 + (long long)seg * a.dim * a.vdim;
          else if (t_end == a.Tn && a.state_out) dst = a.state_out + st0;
          if (dst && row < a.dim && !fail) {
            dst += (long long)row * a.vdim + c * 32;
#pragma unroll
            for (int i = 0; i < 32; i += 4)
              if (c * 32 + i < ne) *reinterpret_cast<float4*>(dst + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
          }
        }
      }
    }
    tc_fence_before();  // the next chunk's products overwrite the columns just read
    if (__syncthreads_or(fail ? 1 : 0)) {
      fail = true;
      break;
    }
    issued = 0;
  }
  if (fail && tid == 0) {
    if (a.status) atomicExch(a.status, *abort_flag ? *abort_flag : 60);
    const uint32_t par = done & 1u;  // give what is in flight a bounded chance to finish
    if (issued >= 1 && !STATE_ONLY) {
      mbar_wait(bar_a, par);
      if (issued == 1) umma_commit(bar_o);
      mbar_wait(bar_o, par);
    }
    if (issued == 2) mbar_wait(bar_s, par);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, 512);
}

template <bool STATE_ONLY>
static size_t rt_smem(int nd, int nv) {
  size_t blocks = 2 * nd + nv;
  if (STATE_ONLY) blocks += nd < 2 ? 1 : 0;  // a key of one block is read as a pair of blocks
  else blocks += 2 * nd + 2 * nv;
  const size_t bytes = blocks * kRtBlock + 1024 + 64 + 1024;
  return bytes < 120 * 1024 ? 120 * 1024 : bytes;  // one CTA owns an SM (it allocates all of TMEM)
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
  p.nd = (a.dim + 63) / 64;
  p.nv = a.vdim > 64 ? 2 : 1;
  p.seg_state = seg_state;
  static bool ready[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) {
    set_error("retention: cudaGetDevice failed");
    return DGPT_E_CUDA;
  }
  if (!ready[dev]) {
    cudaError_t e = cudaFuncSetAttribute(retention_tc_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)rt_smem<true>(2, 2));
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(retention_tc_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)rt_smem<false>(2, 2));
    if (e != cudaSuccess) {
      set_error("retention: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
      return DGPT_E_CUDA;
    }
    ready[dev] = true;
  }
  const int heads = a.n_seq * a.H * p.n_slice;
  if (p.n_seg > 1) {
    retention_tc_kernel<true><<<heads * (p.n_seg - 1), kRtThreads, rt_smem<true>(p.nd, p.nv), st>>>(p);
    if (int e = launch_status("retention_tc (segments)")) return e;
  }
  retention_tc_kernel<false><<<heads * p.n_seg, kRtThreads, rt_smem<false>(p.nd, p.nv), st>>>(p);
  return launch_status("retention_tc");
}

}  // namespace dgpt
