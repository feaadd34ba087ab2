// Attention over cached rows on tcgen05 (sm_100a): one or two persistent CTAs per SM walk through (query row, head group,
// key split) items; the rows of an item pass through shared memory once and serve all its heads.
//
// A tile is 128 keys: dk columns of each row as keys and dv columns as values (the same columns where the cache holds
// latents), cut into units of 128 columns (two 64-column, 128-byte-swizzled blocks, 32 KB; one block where neither keys
// nor values have more than 64 columns).
//   S^T[key, head]    = K Q^T      M = 128 keys,    N = heads, K = dk    A: key units, K-major;            B: Q, K-major
//   O^T[column, head] += V^T P^T   M = 128 columns, N = heads, K = keys  A: a value unit, read MN-major;   B: P, K-major
// so the heads that share a row are the N of both products: 16, 32 or 64 of them cost the same passes over the tile, and
// nothing is padded to 128 rows of queries.  Decode is bound by reading the rows.
//   warp 5, lane 0  loader: Q of the item, then the units of its tiles into a ring, through TMA straight from the pages
//   warp 4, lane 0  issuer: S^T into one of two TMEM buffers, O^T += V^T P^T; with room in the ring the scores of the
//                   next tile are issued before the sums of this one
//   warps 0-3       softmax, one thread per key: probabilities against a running reference per head that only moves when
//                   it is exceeded by 2^8 (found with one barrier vote per tile), written as bf16 into shared memory;
//                   after the item's last tile, one thread per column: normalise, gate, store
// A row of a unit that holds fewer than 64 columns leaves the block's other accumulator rows undefined; they are not read.
// TMEM columns: S0 [0, N)  S1 [N, 2N)  O of unit u [2N + u N, +N).
// Every mbarrier wait is bounded.  When one runs out the abort flag is raised, the loader and the issuer stop and drain
// what they have in flight, the softmax warps run through their remaining tiles without waiting (so that every CTA
// barrier is still met by all of them), TMEM is freed and the status word names the wait.
#include "latent_attn.cuh"
#include "tcgen05.cuh"

namespace dgpt {
namespace tc {

constexpr int kLtKeys = 128;
constexpr uint32_t kLtBlock = kLtKeys * 128;  // [128 keys][64 columns] bf16, swizzled
constexpr uint32_t kLtUnit = 2 * kLtBlock;
constexpr int kLtThreads = 192;
constexpr int kLtMaxUnits = 10;

struct LtParams {
  LatentArgs a;
  int n_rows, n_groups, n_items;  // item = (split * n_groups + group) * n_rows + row
  int per, gpk;                   // heads that share a row, and item groups they make
  int n_units;                    // units in the ring
  uint32_t unit_bytes;
  int uk, uv, upt;                // units of a tile's keys and values (the same ones for latents), and of both
  int align;                      // tiles of a key range start at a multiple of this many slots
  int box;                        // slots per TMA box
};

// blocks of 64 columns in unit u of a vector of `cols` columns
__device__ __forceinline__ int lt_blocks(int cols, int u) { return cols - u * 128 > 64 ? 2 : 1; }

struct LtItem {
  int row, seq, g, h0, nh, split;
  int begin[3], end[3], base[3];  // the slot ranges and where their tiles start
  int n_first, n_second;          // tiles of the first range, of the first two
  int t0, n;                      // this split's tiles
};

// KEPT: the cache holds first keys that are seen from every distance, a slot range of their own
template <bool KEPT>
__device__ __forceinline__ LtItem lt_item(const LtParams& p, int item, int N) {
  LtItem it;
  const int gs = item / p.n_rows;
  it.row = item - gs * p.n_rows;
  it.g = 0;
  it.h0 = 0;
  it.split = gs;
  int first = 0;
  if (p.n_groups > 1) {
    it.split = gs / p.n_groups;
    const int grp = gs - it.split * p.n_groups;
    it.g = grp / p.gpk;
    first = (grp - it.g * p.gpk) * N;
    it.h0 = it.g * p.per + first;
  }
  it.nh = min(N, p.per - first);
  const LatentKeys k = latent_keys(p.a, it.row);
  it.seq = k.seq;
  // [0, ks) and [lo, n), cut where slots change from the first run to the second; the cut lies in one of the two
  const bool own = k.lo >= k.n0;
  it.begin[0] = 0;
  it.end[0] = KEPT ? min(k.ks, k.n0) : 0;
  it.begin[1] = own ? k.s1 : k.lo;
  it.end[1] = own ? (KEPT ? k.s1 + max(0, k.ks - k.n0) : k.s1) : k.n0;
  it.begin[2] = k.s1 + max(0, k.lo - k.n0);
  it.end[2] = k.s1 + (k.n - k.n0);
  int nt[3];
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    it.base[i] = it.begin[i] & ~(p.align - 1);  // a power of two
    nt[i] = it.end[i] > it.begin[i] ? (it.end[i] - it.base[i] + kLtKeys - 1) / kLtKeys : 0;
  }
  it.n_first = KEPT ? nt[0] : 0;
  it.n_second = it.n_first + nt[1];
  const int total = it.n_second + nt[2];
  if (p.a.n_splits == 1) {
    it.t0 = 0;
    it.n = total;
  } else {
    const int per = (total + p.a.n_splits - 1) / p.a.n_splits;
    it.t0 = min(total, it.split * per);
    it.n = min(total, it.t0 + per) - it.t0;
  }
  return it;
}
// first slot of tile j of the item, and the limits of its range
template <bool KEPT>
__device__ __forceinline__ int lt_tile(const LtItem& it, int j, int& begin, int& end) {
  const int t = it.t0 + j;
  if (KEPT && t < it.n_first) {
    begin = it.begin[0];
    end = it.end[0];
    return it.base[0] + t * kLtKeys;
  }
  const bool last = t >= it.n_second;
  begin = last ? it.begin[2] : it.begin[1];
  end = last ? it.end[2] : it.end[1];
  return (last ? it.base[2] : it.base[1]) + (t - (last ? it.n_second : it.n_first)) * kLtKeys;
}

__device__ __forceinline__ void tma_load_3d(uint32_t dst, const CUtensorMap* map, uint32_t bar, int c0, int c1, int c2) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
      ::"r"(dst), "l"(reinterpret_cast<uint64_t>(map)), "r"(bar), "r"(c0), "r"(c1), "r"(c2)
      : "memory");
}
// The four softmax warps: a barrier, and a barrier that tells every thread whether any of them said yes.
__device__ __forceinline__ void lt_sync() { asm volatile("barrier.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ bool lt_any(bool mine) {
  int r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\tsetp.ne.s32 p, %1, 0;\n\tbarrier.red.or.pred q, 2, 128, p;\n\tselp.s32 %0, 1, 0, q;\n\t}"
      : "=r"(r)
      : "r"((int)mine)
      : "memory");
  return r != 0;
}
// op over the 32 lanes for each of 16 values at once: lane l returns the result of value l & 15.  Every step halves the
// values a lane still carries, so 16 shuffles do the work of 80.
template <typename F>
__device__ __forceinline__ float lt_reduce16(const float* v, int lane, F op) {
  float a[8], b[4], c[2];
#pragma unroll
  for (int i = 0; i < 8; ++i) {  // keep values 8 (lane bit 3) + i
    const bool hi = lane & 8;
    const float keep = hi ? v[8 + i] : v[i], send = hi ? v[i] : v[8 + i];
    a[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, 8));
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const bool hi = lane & 4;
    const float keep = hi ? a[4 + i] : a[i], send = hi ? a[i] : a[4 + i];
    b[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, 4));
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const bool hi = lane & 2;
    const float keep = hi ? b[2 + i] : b[i], send = hi ? b[i] : b[2 + i];
    c[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, 2));
  }
  const bool hi = lane & 1;
  const float keep = hi ? c[1] : c[0], send = hi ? c[0] : c[1];
  const float d = op(keep, __shfl_xor_sync(0xffffffffu, send, 1));
  return op(d, __shfl_xor_sync(0xffffffffu, d, 16));
}

// NB: heads per group = 16 NB; HS <= 16 NB: heads the softmax looks after (a group may hold fewer than 16).
// SHARED: a tile's values are its keys (latents), whose cache has no kept first keys.
template <int NB, int HS, bool SHARED>
__global__ void __launch_bounds__(kLtThreads, NB == 4 ? 1 : 2)
latent_tc_kernel(const __grid_constant__ CUtensorMap mq, const __grid_constant__ CUtensorMap mc, const LtParams p) {
  constexpr int N = 16 * NB;
  constexpr uint32_t kIdescS = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(N >> 3) << 17) | (8u << 24);
  constexpr uint32_t kIdescO = kIdescS | (1u << 15);  // A is read MN-major
  constexpr uint32_t kQBlock = N * 128;               // [N heads][64 columns]
  constexpr uint32_t kPBlock = N * 128;               // [N heads][64 keys]
  constexpr uint32_t kTmemCols = NB == 1 ? 128 : (NB == 2 ? 256 : 512);  // N (2 + 4) columns at most
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int UT = p.upt, UK = p.uk, UV = p.uv, NU = p.n_units;
  const int v_unit = SHARED ? 0 : UK;  // where a tile's value units start
  const int nqb = SHARED ? 2 * UK : (p.a.dk + 63) / 64;  // 64-column blocks of Q
  const uint32_t unit_bytes = SHARED ? kLtUnit : p.unit_bytes;
  uint8_t* sU = smem;
  uint8_t* sQ = sU + (size_t)NU * unit_bytes;
  uint8_t* sP = sQ + (size_t)2 * UK * kQBlock;  // one or two buffers of two blocks
  // With room in the ring for the next tile's keys beside a tile the scores of the next tile are issued before the sums
  // of this one, and P needs two buffers; otherwise the next scores follow the sums, and their arrival also says that P has been read.  (Issuing
  // the part of the next scores that the ring could hold before the sums was measured 12 % slower: every change between
  // the two kinds of product costs the tensor pipe more than the wait it fills.)
  const bool ahead = NU >= UT + UK;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + (ahead ? 4 : 2) * kPBlock);
  float* red = reinterpret_cast<float*>(bars + 32);  // [4 warps][N]
  float* fac = red + 4 * N;                          // [4 warps][N]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(fac + 4 * N);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const uint32_t aU = smem_u32(sU), aQ = smem_u32(sQ), aP = smem_u32(sP);
  const uint32_t bar0 = smem_u32(bars);
  const uint32_t bar_q = bar0, bar_qf = bar0 + 8, bar_of = bar0 + 16, bar_drain = bar0 + 24, bar_s = bar0 + 32, bar_p = bar0 + 48,
                 bar_o = bar0 + 64, bar_u = bar0 + 80, bar_uf = bar_u + 8 * kLtMaxUnits;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

  if (tid == 0) {
    *abort_flag = 0;
    for (int i = 0; i < 10 + 2 * kLtMaxUnits; ++i) mbar_init(bar0 + 8 * i, (i == 2 || i == 6 || i == 7) ? 128 : 1);  // O free; P ready
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    fence_async_smem();
  }
  if (warp == 0) {
    tmem_alloc(smem_u32(tmem_slot), kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  dep_wait();

  if (warp == 5) {
    // ================= loader =================
    if (lane == 0) {
      asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&mq)) : "memory");
      asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&mc)) : "memory");
      unsigned un = 0u, items = 0u;  // units and items loaded so far
      bool ok = true;
      const int pt = p.a.kv.page_tokens;
      const LatentArgs& a = p.a;
      for (int item = blockIdx.x; ok && item < p.n_items; item += gridDim.x) {
        const LtItem it = lt_item<!SHARED>(p, item, N);
        if (it.n == 0) continue;
        if (items > 0) ok = wait_or_abort(bar_qf, (items - 1) & 1u, abort_flag, 50);  // the last scores of the item before are done
        if (!ok) break;
        mbar_expect_tx(bar_q, (uint32_t)nqb * kQBlock);
        for (int c = 0; c < nqb; ++c) tma_load_3d(aQ + c * kQBlock, &mq, bar_q, c * 64, it.h0, it.row);
        ++items;
        for (int j = 0; ok && j < it.n; ++j) {
          int begin, end;
          const int slot = lt_tile<!SHARED>(it, j, begin, end);
          const int boxes = min(kLtKeys / p.box, (end - slot + p.box - 1) / p.box);
          for (int u = 0; ok && u < UT; ++u, ++un) {
            const unsigned s = un % (unsigned)NU, round = un / (unsigned)NU;
            if (round > 0) ok = wait_or_abort(bar_uf + 8 * s, (round - 1) & 1u, abort_flag, 51);
            if (!ok) break;
            const uint32_t full = bar_u + 8 * s, dst = aU + s * unit_bytes;
            const bool key = u < UK;
            const int blocks = SHARED ? 2 : key ? lt_blocks(a.dk, u) : lt_blocks(a.dv, u - UK);
            const int col = SHARED ? u * 128 : key ? it.g * a.dk + u * 128 : a.v_col + it.g * a.dv + (u - UK) * 128;
            mbar_expect_tx(full, (uint32_t)boxes * p.box * 128u * blocks);
            for (int b = 0; b < boxes; ++b) {
              const int at = slot + b * p.box;
              int pg = it.seq, in = at;
              if (p.a.kv.page_table) {
                const int lp = at / pt;
                pg = p.a.kv.page_table[(long long)it.seq * p.a.kv.max_pages + lp];
                in = at - lp * pt;
              }
              tma_load_3d(dst + b * p.box * 128, &mc, full, col, in, pg);
              if (blocks == 2) tma_load_3d(dst + kLtBlock + b * p.box * 128, &mc, full, col + 64, in, pg);
            }
          }
        }
      }
      if (!ok || *abort_flag) {  // let the copies in flight land
        if (p.a.status) atomicExch(p.a.status, *abort_flag ? *abort_flag : 50);
        if (items > 0) mbar_wait(bar_q, (items - 1) & 1u);
        for (unsigned i = 0; i < (unsigned)NU && i < un; ++i)
          mbar_wait(bar_u + 8 * ((un - 1 - i) % (unsigned)NU), ((un - 1 - i) / (unsigned)NU) & 1u);
      }
    }
  } else if (warp == 4) {
    // ================= MMA issuer =================
    if (lane == 0) {
      const uint64_t dC = smem_desc(0, 16, 1024), dM = smem_desc(0, kLtBlock, 1024);  // K-major rows; MN-major pairs of blocks
      unsigned g = 0u, items = 0u;  // tiles; items
      bool ok = true;
      for (int item = blockIdx.x; ok && item < p.n_items; item += gridDim.x) {
        const LtItem it = lt_item<!SHARED>(p, item, N);
        if (it.n == 0) continue;
        ok = wait_or_abort(bar_q, items & 1u, abort_flag, 52);
        auto issue_s = [&](unsigned gt, bool last) {
          const uint32_t d = tmem + (gt & 1u) * N;
          for (int u = 0; ok && u < UK; ++u) {
            const unsigned un = gt * (unsigned)UT + (unsigned)u, s = un % (unsigned)NU;
            ok = wait_or_abort(bar_u + 8 * s, (un / (unsigned)NU) & 1u, abort_flag, 53);
            if (!ok) return;
            tc_fence_after();
            const uint64_t da = dC + ((aU + s * unit_bytes) >> 4), db = dC + ((aQ + 2 * u * kQBlock) >> 4);
            if (SHARED || lt_blocks(p.a.dk, u) == 2) umma_ss8<2, kLtBlock / 16, 2, kQBlock / 16>(d, da, db, kIdescS, u > 0 ? 1u : 0u);
            else umma_ss4<2, 2>(d, da, db, kIdescS, u > 0 ? 1u : 0u);
            if (!SHARED) umma_commit(bar_uf + 8 * s);  // keys are done with
          }
          umma_commit(bar_s + 8 * (gt & 1u));
          if (last) umma_commit(bar_qf);
        };
        if (ok) issue_s(g, it.n == 1);
        for (int j = 0; ok && j < it.n; ++j, ++g) {
          const unsigned b = g & 1u;
          if (ahead && j + 1 < it.n) issue_s(g + 1, j + 2 == it.n);
          ok = ok && wait_or_abort(bar_p + 8 * b, (g >> 1) & 1u, abort_flag, 54);
          if (ok && j == 0 && items > 0) ok = wait_or_abort(bar_of, (items - 1) & 1u, abort_flag, 55);  // the last item's O has been read
          if (!ok) break;
          tc_fence_after();
          for (int u = 0; u < UV; ++u) {
            const unsigned un = g * (unsigned)UT + (unsigned)(v_unit + u), s = un % (unsigned)NU;
            if (!SHARED) {
              ok = wait_or_abort(bar_u + 8 * s, (un / (unsigned)NU) & 1u, abort_flag, 53);
              if (!ok) break;
              tc_fence_after();
            }
            umma_ss8<128, 512, 2, kPBlock / 16>(tmem + 2 * N + u * N, dM + ((aU + s * unit_bytes) >> 4), dC + ((aP + (ahead ? 2 * b * kPBlock : 0u)) >> 4),
                                            kIdescO, j > 0 ? 1u : 0u);
            umma_commit(bar_uf + 8 * s);
          }
          if (!ok) break;
          umma_commit(bar_o + 8 * b);
          if (!ahead && j + 1 < it.n) issue_s(g + 1, j + 2 == it.n);
        }
        ++items;
      }
      if (!ok || *abort_flag) {
        if (p.a.status) atomicExch(p.a.status, *abort_flag ? *abort_flag : 52);
        umma_commit(bar_drain);  // completes when everything issued so far has finished
        mbar_wait(bar_drain, 0);
      }
    }
  } else {
    // ================= softmax: one thread per key; one thread per column at the end =================
    const uint32_t lane_addr = tmem + ((uint32_t)(warp * 32) << 16);
    unsigned g = 0u;
    bool fail = false;
    const long long RH = (long long)p.n_rows * p.a.H;
    if (HS < N) {  // heads nobody looks after: their probabilities are zeros, once
      for (int i = tid; i < (int)((ahead ? 4 : 2) * kPBlock / 16); i += 128) reinterpret_cast<uint4*>(sP)[i] = make_uint4(0u, 0u, 0u, 0u);
      lt_sync();
    }
    for (int item = blockIdx.x; item < p.n_items; item += gridDim.x) {
      const LtItem it = lt_item<!SHARED>(p, item, N);
      const int nh = it.nh;
      constexpr int HL = (N + 31) / 32;  // heads a lane looks after at the end of the item
      float gate[HL];
#pragma unroll
      for (int c = 0; c < HL; ++c) {  // wanted at the end only
        const int h = lane + 32 * c;
        gate[c] = 1.f;
        if (p.a.gate && h < nh)
          gate[c] = __bfloat162float(static_cast<const __nv_bfloat16*>(p.a.gate)[(long long)it.row * p.a.gate_rs + it.h0 + h]);
      }
      float m[HS], l[HS];
#pragma unroll
      for (int h = 0; h < HS; ++h) {
        m[h] = -INFINITY;
        l[h] = 0.f;
      }
      for (int j = 0; j < it.n; ++j, ++g) {
        const unsigned b = g & 1u;
        int begin, end;
        const int slot = lt_tile<!SHARED>(it, j, begin, end) + tid;
        if (!fail && !wait_or_abort(bar_s + 8 * b, (g >> 1) & 1u, abort_flag, 56)) fail = true;
        fail = __any_sync(0xffffffffu, fail);
        tc_fence_after();
        const bool seen = slot >= begin && slot < end;
        if (!fail && slot >= end) {  // nothing was loaded here, or rows nobody has written: 0 * x must stay 0
          for (int u = 0; u < UV; ++u) {
            const unsigned un = g * (unsigned)UT + (unsigned)(v_unit + u), us = un % (unsigned)NU;
            if (!SHARED && !wait_or_abort(bar_u + 8 * us, (un / (unsigned)NU) & 1u, abort_flag, 59)) break;  // still on its way
            uint8_t* unit = sU + (size_t)us * unit_bytes;
            const bool two = SHARED || lt_blocks(p.a.dv, u) == 2;
#pragma unroll
            for (int c = 0; c < 8; ++c) {
              reinterpret_cast<uint4*>(unit + tid * 128)[c] = make_uint4(0u, 0u, 0u, 0u);
              if (two) reinterpret_cast<uint4*>(unit + kLtBlock + tid * 128)[c] = make_uint4(0u, 0u, 0u, 0u);
            }
          }
        }
        float s[N];
#pragma unroll
        for (int c = 0; c < NB; ++c) tmem_ld16_nowait(lane_addr + b * N + c * 16, s + 16 * c);
        tc_wait_ld();
        bool over = false;
#pragma unroll
        for (int h = 0; h < HS; ++h) {
          s[h] = seen ? s[h] * p.a.scale_log2 : -INFINITY;
          over |= s[h] > m[h] + 8.f;
        }
        if (lt_any(over && !fail)) {  // some head's reference has to move: the tile's maxima, the same in every thread
#pragma unroll
          for (int h = HS; h < N; ++h) s[h] = -INFINITY;
#pragma unroll
          for (int c = 0; c < NB; ++c) {
            const float t = lt_reduce16(s + 16 * c, lane, [](float x, float y) { return fmaxf(x, y); });
            if (lane < 16) red[warp * N + 16 * c + lane] = t;
          }
          lt_sync();
          float alpha[N];
#pragma unroll
          for (int h = HS; h < N; ++h) alpha[h] = 1.f;
#pragma unroll
          for (int h = 0; h < HS; ++h) {
            const float mn = fmaxf(fmaxf(fmaxf(red[h], red[N + h]), fmaxf(red[2 * N + h], red[3 * N + h])), m[h]);
            alpha[h] = mn == -INFINITY ? 1.f : ex2(m[h] - mn);  // -inf before the first tile: 0
            m[h] = mn;
            l[h] *= alpha[h];
          }
          if (j > 0) {
            // O may only be touched when no product is in flight on it: the tile before must be done, and this tile's
            // waits for this thread's arrival below
            if (!fail && !wait_or_abort(bar_o + 8 * (b ^ 1u), ((g - 1) >> 1) & 1u, abort_flag, 57)) fail = true;
            fail = __any_sync(0xffffffffu, fail);
            tc_fence_after();
            for (int u = 0; u < UV; ++u) {
#pragma unroll
              for (int c = 0; c < NB; ++c) {
                float v[16];
                const uint32_t addr = lane_addr + 2 * N + u * N + c * 16;
                tmem_ld16_nowait(addr, v);
                tc_wait_ld();
                uint32_t w[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) w[i] = __float_as_uint(v[i] * alpha[16 * c + i]);
                tmem_st16(addr, w);
              }
            }
            tc_wait_st();
          }
          lt_sync();  // `red` may be written again
        }
        uint8_t* pb = sP + ((ahead ? 2 * b : 0u) + (tid >> 6)) * kPBlock + (tid & 7) * 2;
        const int chunk = (tid & 63) >> 3;
#pragma unroll
        for (int h = 0; h < HS; ++h) {
          const float e = ex2(s[h] - m[h]);  // not seen: 0 (m is finite: every tile holds a key that is seen)
          l[h] += e;
          *reinterpret_cast<__nv_bfloat16*>(pb + h * 128 + ((chunk ^ (h & 7)) << 4)) = __float2bfloat16_rn(e);
        }
        fence_async_smem();
        tc_fence_before();
        mbar_arrive(bar_p + 8 * b);
      }
      // ---- the item's result ----
      if (it.n > 0) {
        const unsigned last = g - 1u;
        if (!fail && !wait_or_abort(bar_o + 8 * (last & 1u), (last >> 1) & 1u, abort_flag, 58)) fail = true;
        fail = __any_sync(0xffffffffu, fail);
        tc_fence_after();
      }
#pragma unroll
      for (int c = 0; c < NB; ++c) {
        float ls[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) ls[i] = 16 * c + i < HS ? l[(16 * c + i) % HS] : 0.f;
        const float t = lt_reduce16(ls, lane, [](float x, float y) { return x + y; });
        if (lane < 16) red[warp * N + 16 * c + lane] = t;
      }
      lt_sync();
      const long long rh0 = (long long)it.row * p.a.H + it.h0;
      const long long slot0 = (long long)it.split * RH + rh0;
      // lane h: 1 / sum and gate of head h, or the sum itself for a split
#pragma unroll
      for (int c = 0; c < HL; ++c) {
        const int h = lane + 32 * c;
        if (h < N) {
          const float sum = (red[h] + red[N + h]) + (red[2 * N + h] + red[3 * N + h]);
          float f = sum > 0.f ? 1.f / sum : 0.f;
          if (p.a.gate) f *= 1.f / (1.f + __expf(-gate[c]));
          fac[warp * N + h] = f;
          if (p.a.n_splits > 1 && warp == 0 && h < nh) p.a.ws_ml[2 * (slot0 + h) + 1] = sum;
        }
      }
      if (p.a.n_splits > 1 && tid == 0) {
#pragma unroll
        for (int h = 0; h < HS; ++h)
          if (h < nh) p.a.ws_ml[2 * (slot0 + h)] = m[h];
      }
      lt_sync();  // `red` may be written again, `fac` is complete
      if (it.n > 0) {
        for (int u = 0; u < UV; ++u) {
          const int col = u * 128 + tid;
#pragma unroll
          for (int c = 0; c < NB; ++c) {
            float v[16];
            tmem_ld16_nowait(lane_addr + 2 * N + u * N + c * 16, v);
            tc_wait_ld();
            if (u == UV - 1 && c == NB - 1) {
              tc_fence_before();
              mbar_arrive(bar_of);  // the next item may overwrite O
            }
            if (p.a.n_splits > 1) {
              if (col < p.a.dv) {
#pragma unroll
                for (int i = 0; i < 16; ++i)
                  if (16 * c + i < nh) p.a.ws_o[(slot0 + 16 * c + i) * p.a.dv + col] = v[i];
              }
              continue;
            }
            // two columns of one head per store: an even lane takes the even head of a pair, its neighbour the odd one
            // (dv is a multiple of 8, so both columns exist or neither does)
            const bool odd = lane & 1;
            __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.a.out) + (long long)it.row * p.a.out_rs + (long long)it.h0 * p.a.dv + (col & ~1);
#pragma unroll
            for (int i = 0; i < 16; i += 2) {
              const float x = v[i] * fac[warp * N + 16 * c + i], y = v[i + 1] * fac[warp * N + 16 * c + i + 1];
              const float got = __shfl_xor_sync(0xffffffffu, odd ? x : y, 1);
              const int h = 16 * c + i + (odd ? 1 : 0);
              if (h < nh && col < p.a.dv)
                *reinterpret_cast<__nv_bfloat162*>(dst + (long long)h * p.a.dv) = odd ? __floats2bfloat162_rn(got, y) : __floats2bfloat162_rn(x, got);
            }
          }
        }
      } else if (p.a.n_splits == 1) {  // no keys at all
        for (int u = 0; u < UV; ++u) {
          const int col = u * 128 + tid;
          for (int h = 0; h < nh && col < p.a.dv; ++h)
            static_cast<__nv_bfloat16*>(p.a.out)[(long long)it.row * p.a.out_rs + (long long)(it.h0 + h) * p.a.dv + col] = __float2bfloat16_rn(0.f);
        }
      }
    }
    if (fail && p.a.status && tid == 0) atomicExch(p.a.status, *abort_flag ? *abort_flag : 56);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, kTmemCols);
}

static bool encode_3d(CUtensorMap* map, const void* base, const cuuint64_t (&dims)[3], const cuuint64_t (&strides)[2],
                      const cuuint32_t (&box)[3]) {
  const cuuint32_t ones[3] = {1, 1, 1};
  CUresult r = encode_fn()(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, ones,
                           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) {
    set_error("latent_attn: cuTensorMapEncodeTiled failed with %d", (int)r);
    return false;
  }
  return true;
}

// heads per group (per = heads that share a row), and what fits beside Q and P in the shared memory (limit: opt-in bytes per CTA)
static int lt_heads(int per) { return per <= 16 ? 16 : (per <= 32 ? 32 : 64); }
struct LtShape {
  int N, uk, uv, upt;
  uint32_t unit_bytes;
  size_t bytes(int units) const {
    return (size_t)2 * uk * N * 128 + (size_t)(units >= upt + uk ? 4 : 2) * N * 128 + 256 + (size_t)32 * N + 64 + 1024 + (size_t)units * unit_bytes +
           (unit_bytes < kLtUnit ? kLtBlock : 0);  // a value unit of one block is read as a pair of blocks: the last one's partner must exist
  }
  int units(size_t limit) const {
    int n = kLtMaxUnits;
    while (n > 0 && bytes(n) > limit) --n;
    return n;
  }
};
static LtShape lt_shape(const LatentArgs& a) {
  LtShape s;
  s.N = lt_heads(a.H / a.G);
  s.uk = (a.dk + 127) / 128;
  s.uv = (a.dv + 127) / 128;
  s.upt = a.v_col == 0 ? s.uk : s.uk + s.uv;
  s.unit_bytes = a.v_col != 0 && a.dk <= 64 && a.dv <= 64 ? kLtBlock : kLtUnit;
  return s;
}

template <int NB, int HS, bool SHARED>
static int lt_launch(const CUtensorMap& mq, const CUtensorMap& mc, const LtParams& p, int grid, size_t smem, cudaStream_t st) {
  cudaError_t e = cudaFuncSetAttribute(latent_tc_kernel<NB, HS, SHARED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) {
    set_error("latent_attn: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
    return DGPT_E_CUDA;
  }
  launch_dep(latent_tc_kernel<NB, HS, SHARED>, dim3(grid), dim3(kLtThreads), smem, st, mq, mc, p);
  return launch_status("latent_attn");
}

static void lt_device(int* sms, int* smem) {
  static int n_sm[64] = {}, n_smem[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) dev = 0;
  if (n_sm[dev] == 0) {
    cudaDeviceGetAttribute(&n_smem[dev], cudaDevAttrMaxSharedMemoryPerBlockOptin, dev);
    cudaDeviceGetAttribute(&n_sm[dev], cudaDevAttrMultiProcessorCount, dev);
  }
  *sms = n_sm[dev] > 0 ? n_sm[dev] : 1;
  *smem = n_smem[dev];
}

}  // namespace tc

bool latent_tc_supported(const LatentArgs& a, const dgpt_kv_layout& kv, int dtype) {
  if (dtype != DGPT_BF16 || a.dk > 512 || a.dv > 512) return false;
  const int pt = kv.page_tokens;
  if (kv.page_table && !((pt >= tc::kLtKeys && pt % tc::kLtKeys == 0) || (pt >= 8 && pt < tc::kLtKeys && tc::kLtKeys % pt == 0))) return false;
  if (kv.page_stride <= 0 || a.q_rs <= 0) return false;
  if (!tc::device_is_sm100() || tc::encode_fn() == nullptr) return false;
  int sms, smem;
  tc::lt_device(&sms, &smem);
  const tc::LtShape sh = tc::lt_shape(a);
  return sh.units((size_t)smem) >= sh.upt;
}

int latent_tc_launch(const LatentArgs& a, const dgpt_kv_layout& kv, cudaStream_t st) {
  using namespace tc;
  int sms, limit;
  lt_device(&sms, &limit);
  const LtShape sh = lt_shape(a);
  const int N = sh.N;
  LtParams p;
  p.a = a;
  p.per = a.H / a.G;
  p.gpk = (p.per + N - 1) / N;
  p.n_rows = a.n_seq * a.Tn;
  p.n_groups = a.G * p.gpk;
  p.n_items = p.n_rows * p.n_groups * a.n_splits;
  p.uk = sh.uk;
  p.uv = sh.uv;
  p.upt = sh.upt;
  p.unit_bytes = sh.unit_bytes;
  // Two CTAs per SM where half the shared memory holds a tile and a unit: while one waits for its scores or its
  // probabilities, the other has products to run.  (NB = 4 needs the registers of a whole SM.)
  int per_sm = 1;
  p.n_units = sh.units((size_t)limit);
  if (N < 64 && p.n_items > sms) {
    const int half = sh.units((size_t)(limit - 1024) / 2);  // each CTA costs another KB of the SM's 228
    if (half > p.upt) {
      per_sm = 2;
      p.n_units = half;
    }
  }
  const int pt = kv.page_tokens;
  p.box = kv.page_table && pt < kLtKeys ? pt : kLtKeys;
  p.align = kv.page_table ? p.box : 1;  // a dense run may be entered at any slot
  CUtensorMap mq, mc;
  {
    const cuuint64_t dims[3] = {(cuuint64_t)a.dk, (cuuint64_t)a.H, (cuuint64_t)p.n_rows};
    const cuuint64_t strides[2] = {(cuuint64_t)a.dk * 2, (cuuint64_t)a.q_rs * 2};
    const cuuint32_t box[3] = {64, (cuuint32_t)N, 1};
    if (!encode_3d(&mq, a.q, dims, strides, box)) return DGPT_E_CUDA;
  }
  {
    const cuuint64_t n_pages = kv.page_table ? (kv.n_pages > 0 ? (cuuint64_t)kv.n_pages : (cuuint64_t)1 << 24) : (cuuint64_t)a.n_seq;
    const cuuint64_t dims[3] = {(cuuint64_t)a.row_w, (cuuint64_t)pt, n_pages};
    const cuuint64_t strides[2] = {(cuuint64_t)a.row_w * 2, (cuuint64_t)kv.page_stride * 2};
    const cuuint32_t box[3] = {64, (cuuint32_t)p.box, 1};
    if (!encode_3d(&mc, kv.k_base, dims, strides, box)) return DGPT_E_CUDA;
  }
  const size_t smem = sh.bytes(p.n_units);
  const int grid = p.n_items < per_sm * sms ? p.n_items : per_sm * sms;
  if (a.v_col == 0) {
    if (N == 16) return lt_launch<1, 16, true>(mq, mc, p, grid, smem, st);
    if (N == 32) return lt_launch<2, 32, true>(mq, mc, p, grid, smem, st);
    return lt_launch<4, 64, true>(mq, mc, p, grid, smem, st);
  }
  if (p.per <= 4) return lt_launch<1, 4, false>(mq, mc, p, grid, smem, st);
  if (p.per <= 8) return lt_launch<1, 8, false>(mq, mc, p, grid, smem, st);
  if (N == 16) return lt_launch<1, 16, false>(mq, mc, p, grid, smem, st);
  if (N == 32) return lt_launch<2, 32, false>(mq, mc, p, grid, smem, st);
  return lt_launch<4, 64, false>(mq, mc, p, grid, smem, st);
}

}  // namespace dgpt
