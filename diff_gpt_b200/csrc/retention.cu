// Retention: linear attention with a fixed decay per head, the recurrent form.
//
//   S_t = decay S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t        per head; q, k rotated (rotate-half pairs), k scaled; S fp32
//
//   retention_decode_kernel   one token per sequence: the state is read and written once (that is what bounds decoding),
//                             rotation, head norm and output gate in the same launch
//   retention_scan_kernel     any sizes, any number of tokens: the state stays in shared memory, tokens one after the other
//   head_norm_gate_kernel     y = rms_norm(o) * silu(g) per head, after the kernels that leave o in fp32
//
// The chunked tensor-core form for prompts is in retention_tc.cu.
#include "retention.cuh"
#include "rowvec.cuh"

namespace dgpt {

constexpr int kRetThreads = 256;

// dst[0..dim) = the rotated vector times `scale`; src: one head's q or k
template <typename T>
__device__ __forceinline__ void rotate_head(const T* __restrict__ src, const float2* __restrict__ cs, int rot, int dim, float scale,
                                            float* dst, int first, int step) {
  const int half = rot >> 1;
  for (int i = first; i < dim; i += step) {
    if (i < half) {
      const float2 c = cs[i];
      const float u = Io<T>::ld(src + i), v = Io<T>::ld(src + i + half);
      dst[i] = (u * c.x - v * c.y) * scale;
      dst[i + half] = (v * c.x + u * c.y) * scale;
    } else if (i >= rot) {
      dst[i] = Io<T>::ld(src + i) * scale;
    }
  }
}

__device__ __forceinline__ float silu_value(float z) { return z / (1.f + expf(-z)); }

// ---- one token per sequence ------------------------------------------------------------------
// CTA per (sequence, head).  Thread groups of vdim / 4 threads take the state's rows in turn, four columns per thread.
template <typename T>
__global__ void __launch_bounds__(kRetThreads) retention_decode_kernel(const RetentionArgs a) {
  extern __shared__ __align__(16) float ret_smem[];
  const int dim = a.dim, e = a.vdim, cols = e >> 2;
  const int groups = kRetThreads / cols;
  float* sq = ret_smem;             // [dim]
  float* sk = sq + a.dim_pad;       // [dim]
  float* so = sk + a.dim_pad;       // [groups][vdim]
  __shared__ float scratch[40];
  const int h = blockIdx.x % a.H, s = blockIdx.x / a.H, tid = threadIdx.x;
  const int g = tid / cols, c = (tid - g * cols) * 4;
  const bool work = g < groups;
  const long long base = ((long long)s * a.H + h) * dim * e + c;
  const float* in = a.state_in + base;
  float* out = a.state_out + base;
  // the first rows of the state are on their way while q and k are rotated
  constexpr int U = 8;
  float4 r[U];
#pragma unroll
  for (int u = 0; u < U; ++u)
    if (work && g + u * groups < dim) r[u] = *reinterpret_cast<const float4*>(in + (long long)(g + u * groups) * e);
  const int pos = a.pos0[s] + (a.step_ptr ? *a.step_ptr : 0);
  const bool ok = pos >= 0 && pos < a.table_len;
  if (!ok && tid == 0 && a.status) *a.status = 1;
  const float2* cs = a.table + (long long)(ok ? pos : 0) * (a.rot >> 1);
  const T* row = static_cast<const T*>(a.in) + (long long)s * a.in_rs;
  FVec<4> v;
  if (work) v = ldt<T, 4>(row + a.v_col + h * e + c);
  const bool mine = tid < cols;
  if (tid < 128) rotate_head<T>(row + a.q_col + h * dim, cs, a.rot, dim, 1.f, sq, tid, 128);
  else rotate_head<T>(row + a.k_col + h * dim, cs, a.rot, dim, a.k_scale, sk, tid - 128, 128);
  const float decay = a.decay[h];
  __syncthreads();
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  if (work) {
    for (int d = g; d < dim; d += U * groups) {
      if (d != g) {
#pragma unroll
        for (int u = 0; u < U; ++u)
          if (d + u * groups < dim) r[u] = *reinterpret_cast<const float4*>(in + (long long)(d + u * groups) * e);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = d + u * groups;
        if (i < dim) {
          const float kd = sk[i], qd = sq[i];
          r[u].x = fmaf(decay, r[u].x, kd * v.v[0]);
          r[u].y = fmaf(decay, r[u].y, kd * v.v[1]);
          r[u].z = fmaf(decay, r[u].z, kd * v.v[2]);
          r[u].w = fmaf(decay, r[u].w, kd * v.v[3]);
          *reinterpret_cast<float4*>(out + (long long)i * e) = r[u];
          acc[0] = fmaf(qd, r[u].x, acc[0]);
          acc[1] = fmaf(qd, r[u].y, acc[1]);
          acc[2] = fmaf(qd, r[u].z, acc[2]);
          acc[3] = fmaf(qd, r[u].w, acc[3]);
        }
      }
    }
    *reinterpret_cast<float4*>(so + g * e + c) = make_float4(acc[0], acc[1], acc[2], acc[3]);
  }
  __syncthreads();
  float o[4] = {0.f, 0.f, 0.f, 0.f};
  float ss = 0.f;
  if (mine) {
    for (int i = 0; i < groups; ++i) {
      const float4 p = *reinterpret_cast<const float4*>(so + i * e + c);
      o[0] += p.x;
      o[1] += p.y;
      o[2] += p.z;
      o[3] += p.w;
    }
    ss = o[0] * o[0] + o[1] * o[1] + o[2] * o[2] + o[3] * o[3];
  }
  const float inv = rsqrtf(block_sum(ss, scratch) / (float)e + a.eps);
  if (mine) {
    const FVec<4> gv = ldt<T, 4>(row + a.g_col + h * e + c);
    FVec<4> y;
#pragma unroll
    for (int i = 0; i < 4; ++i) y.v[i] = o[i] * inv * silu_value(gv.v[i]);
    stt<T, 4>(static_cast<T*>(a.y) + (long long)s * a.y_rs + h * e + c, y);
  }
}

// ---- any sizes, token by token ------------------------------------------------------------------
// CTA per (sequence, head, slice of `es` value columns); the slice of the state lives in shared memory.
template <typename T>
__global__ void __launch_bounds__(kRetThreads) retention_scan_kernel(const RetentionArgs a, int es) {
  extern __shared__ __align__(16) float ret_smem[];
  const int dim = a.dim, e0 = blockIdx.y * es, ne = min(es, a.vdim - e0);
  float* S = ret_smem;                            // [dim][es]
  float* sq = S + (size_t)dim * es;               // [dim]
  float* sk = sq + a.dim_pad;                     // [dim]
  float* part = sk + a.dim_pad;                   // [row groups][ne]
  const int h = blockIdx.x % a.H, s = blockIdx.x / a.H, tid = threadIdx.x;
  const int step = a.step_ptr ? *a.step_ptr : 0;
  const float decay = a.decay[h];
  const long long base = ((long long)s * a.H + h) * dim * a.vdim + e0;
  const int groups = max(1, kRetThreads / ne);  // rows of the state worked on at a time
  for (int i = tid; i < dim * ne; i += kRetThreads) {
    const int d = i / ne, c = i - d * ne;
    S[d * es + c] = a.state_in ? a.state_in[base + (long long)d * a.vdim + c] : 0.f;
  }
  for (int t = 0; t < a.Tn; ++t) {
    const long long tok = (long long)s * a.Tn + t;
    const int pos = a.pos0[s] + step + t;
    const bool ok = pos >= 0 && pos < a.table_len;
    if (!ok && tid == 0 && a.status) *a.status = 1;
    const float2* cs = a.table + (long long)(ok ? pos : 0) * (a.rot >> 1);
    const T* row = static_cast<const T*>(a.in) + tok * a.in_rs;
    __syncthreads();  // the last token's vectors and partial sums have been read
    if (tid < 128) rotate_head<T>(row + a.q_col + h * dim, cs, a.rot, dim, 1.f, sq, tid, 128);
    else rotate_head<T>(row + a.k_col + h * dim, cs, a.rot, dim, a.k_scale, sk, tid - 128, 128);
    __syncthreads();
    for (int i = tid; i < groups * ne; i += kRetThreads) {
      const int g = i / ne, c = i - g * ne;
      const float v = Io<T>::ld(row + a.v_col + h * a.vdim + e0 + c);
      float acc = 0.f;
      for (int d = g; d < dim; d += groups) {
        const float x = fmaf(decay, S[d * es + c], sk[d] * v);
        S[d * es + c] = x;
        acc = fmaf(sq[d], x, acc);
      }
      part[g * ne + c] = acc;
    }
    __syncthreads();
    for (int c = tid; c < ne; c += kRetThreads) {
      float o = 0.f;
      for (int g = 0; g < groups; ++g) o += part[g * ne + c];
      a.o[tok * a.H * a.vdim + h * a.vdim + e0 + c] = o;
    }
  }
  __syncthreads();
  if (a.state_out) {
    for (int i = tid; i < dim * ne; i += kRetThreads) {
      const int d = i / ne, c = i - d * ne;
      a.state_out[base + (long long)d * a.vdim + c] = S[d * es + c];
    }
  }
}

// One warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* __restrict__ o, const T* __restrict__ gate, long long g_rs,
                                                             float eps, T* __restrict__ y, long long y_rs, long long n, int H, int e) {
  const long long w = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (w >= n * H) return;
  const long long tok = w / H;
  const int h = (int)(w - tok * H), lane = threadIdx.x & 31;
  const float* src = o + w * e;
  float ss = 0.f;
  for (int c = lane; c < e; c += 32) ss += src[c] * src[c];
  const float inv = rsqrtf(warp_sum(ss) / (float)e + eps);
  for (int c = lane; c < e; c += 32)
    Io<T>::st(y + tok * y_rs + h * e + c, src[c] * inv * silu_value(Io<T>::ld(gate + tok * g_rs + h * e + c)));
}

static int ret_max_smem() {
  static int bytes[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return 0;
  if (bytes[dev] == 0) cudaDeviceGetAttribute(&bytes[dev], cudaDevAttrMaxSharedMemoryPerBlockOptin, dev);
  return bytes[dev];
}

template <typename T>
static int head_norm_gate(const RetentionArgs& a, cudaStream_t st) {
  const long long n = (long long)a.n_seq * a.Tn;
  head_norm_gate_kernel<T><<<(unsigned)((n * a.H + 7) / 8), 256, 0, st>>>(a.o, static_cast<const T*>(a.in) + a.g_col, a.in_rs, a.eps,
                                                                          static_cast<T*>(a.y), a.y_rs, n, a.H, a.vdim);
  return launch_status("head_norm_gate");
}

template <typename T>
static int retention_recurrent(const RetentionArgs& a, cudaStream_t st) {
  const int e = a.vdim;
  auto vec_ok = [&](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool fused = a.Tn == 1 && a.state_in && a.state_out && e % 4 == 0 && e <= 4 * kRetThreads && a.dim <= 4096 && a.in_rs % 4 == 0 &&
                     a.v_col % 4 == 0 && a.g_col % 4 == 0 && a.y_rs % 4 == 0 && vec_ok(a.in) && vec_ok(a.y) && vec_ok(a.state_in) &&
                     vec_ok(a.state_out);
  if (fused) {
    const int groups = kRetThreads / (e / 4);
    const size_t smem = ((size_t)2 * a.dim_pad + (size_t)groups * e) * 4;
    retention_decode_kernel<T><<<(unsigned)(a.n_seq * a.H), kRetThreads, smem, st>>>(a);
    return launch_status("retention_decode");
  }
  // the widest slice of value columns whose state fits; a few CTAs per head are welcome while there are few heads
  const size_t limit = (size_t)ret_max_smem();
  auto need = [&](int es) { return ((size_t)a.dim * es + 2 * (size_t)a.dim_pad + (size_t)(es > kRetThreads ? es : kRetThreads)) * 4; };
  int es = e;
  while (es > 1 && (need(es) > limit || (es > 32 && (long long)a.n_seq * a.H * ((e + es - 1) / es) < 148))) es = (es + 1) / 2;
  if (need(es) > limit) {
    set_error("retention: a key size of %d does not fit the shared memory", a.dim);
    return DGPT_E_UNSUPPORTED;
  }
  cudaError_t err = cudaFuncSetAttribute(retention_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)need(es));
  if (err != cudaSuccess) {
    set_error("retention: cudaFuncSetAttribute: %s", cudaGetErrorString(err));
    return DGPT_E_CUDA;
  }
  const dim3 grid((unsigned)(a.n_seq * a.H), (unsigned)((e + es - 1) / es));
  retention_scan_kernel<T><<<grid, kRetThreads, need(es), st>>>(a, es);
  if (int x = launch_status("retention_scan")) return x;
  return head_norm_gate<T>(a, st);
}

constexpr int kRetChunkMin = 16;  // tokens per sequence from which the chunked form is faster than walking through them

}  // namespace dgpt

using namespace dgpt;

extern "C" int dgpt_retention(const void* in, int64_t in_row_stride, int32_t q_col, int32_t k_col, int32_t v_col, int32_t g_col,
                              const float* table, int32_t table_len, int32_t rot_dims, const int32_t* pos0, const int32_t* step_ptr,
                              const float* decay, float min_decay, float k_scale, const float* state_in, float* state_out,
                              float eps, void* y, int64_t y_row_stride, float* workspace, size_t workspace_bytes, int32_t n_seq, int32_t T, int32_t H,
                              int32_t dim, int32_t vdim, int32_t dtype, int32_t impl, int32_t* status, void* stream) {
  DGPT_REQUIRE(in && table && pos0 && decay && y, "retention: NULL pointer");
  DGPT_REQUIRE(n_seq >= 0 && T >= 0 && H > 0 && dim > 0 && vdim > 0 && rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim && table_len > 0,
               "retention: bad sizes");
  DGPT_REQUIRE((long long)n_seq * H <= 0x7fffffff, "retention: too many sequences");
  DGPT_REQUIRE(q_col >= 0 && k_col >= 0 && v_col >= 0 && g_col >= 0, "retention: bad columns");
  DGPT_REQUIRE(state_in == nullptr || state_in != state_out || T <= 1, "retention: the state may be updated in place for T = 1 only");
  DGPT_REQUIRE(dtype == DGPT_F32 || dtype == DGPT_BF16, "retention: unknown dtype %d", dtype);
  DGPT_REQUIRE(impl >= 0 && impl <= 2, "retention: impl must be 0 (auto), 1 (recurrent) or 2 (chunks on tcgen05)");
  if (n_seq == 0 || T == 0) return DGPT_OK;
  RetentionArgs a;
  a.in = in; a.in_rs = in_row_stride;
  a.q_col = q_col; a.k_col = k_col; a.v_col = v_col; a.g_col = g_col;
  a.table = reinterpret_cast<const float2*>(table); a.table_len = table_len; a.rot = rot_dims;
  a.pos0 = pos0; a.step_ptr = step_ptr;
  a.decay = decay; a.k_scale = k_scale;
  a.state_in = state_in; a.state_out = state_out;
  a.eps = eps;
  a.y = y; a.y_rs = y_row_stride;
  a.o = workspace;
  a.n_seq = n_seq; a.Tn = T; a.H = H; a.dim = dim; a.vdim = vdim;
  a.dim_pad = (dim + 3) / 4 * 4;
  a.status = status;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const size_t need = dgpt_retention_workspace_bytes(n_seq, T, H, dim, vdim);
  if (workspace == nullptr || workspace_bytes < need || (reinterpret_cast<uintptr_t>(workspace) & 15) != 0) {
    set_error("retention: a 16-byte aligned workspace of %zu bytes is needed, %zu given", need, workspace_bytes);
    return DGPT_E_WORKSPACE;
  }
  const bool tc_ok = retention_tc_supported(a, dtype, min_decay);
  if (impl == 2 && !tc_ok) {
    set_error("retention: the chunked form covers bf16 with key sizes up to 128, sizes and columns that are multiples of 8 and decays "
              "from 1/16 on (dtype %d, sizes %d and %d, smallest decay %g)", dtype, dim, vdim, (double)min_decay);
    return DGPT_E_UNSUPPORTED;
  }
  if (tc_ok && (impl == 2 || (impl == 0 && T >= kRetChunkMin))) {
    const size_t o_bytes = ((size_t)n_seq * T * H * vdim * sizeof(float) + 15) & ~(size_t)15;
    if (int e = retention_tc_launch(a, workspace + o_bytes / sizeof(float), st)) return e;
    return vdim > 128 ? head_norm_gate<__nv_bfloat16>(a, st) : DGPT_OK;
  }
  return dtype == DGPT_F32 ? retention_recurrent<float>(a, st) : retention_recurrent<__nv_bfloat16>(a, st);
}

extern "C" size_t dgpt_retention_workspace_bytes(int32_t n_seq, int32_t T, int32_t H, int32_t dim, int32_t vdim) {
  if (n_seq <= 0 || T <= 0 || H <= 0 || dim <= 0 || vdim <= 0) return 16;
  // o where it waits for its norm, then the states of the chunked form's segments
  return ((((size_t)n_seq * T * H * vdim * sizeof(float)) + 15) & ~(size_t)15) + retention_tc_workspace_bytes(n_seq, T, H, dim, vdim);
}
