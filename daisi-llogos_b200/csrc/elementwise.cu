// Memory-bound kernels of the decoder: embedding rows, residual add + RMSNorm,
// query/key preparation (per-head norm, bias, rotation, cache write), SiLU-gating,
// cache writes and small index updates.  All statistics and the residual stream are
// float32; activations are float32 or bfloat16.
//
// Counterparts in the reference (formulas only): Daisi.Llogos.Cuda/kernels/elementwise.cu
// rms_norm :18-48, add_rms_norm_residual :703-733, rope :243-290, swiglu :942-950,
// embedding_lookup :402-457; kernels/composite_ops.cu per_head_rms_norm :106-136,
// kv_cache_write :198-224.
#include "common.cuh"
#include "kernel_args.h"

LLG_API const char* llg_last_error() { return g_llg_error; }
LLG_API int llg_page_size() { return LLG_PAGE; }

// ---- embedding ----------------------------------------------------------------------

template <typename TT>
__global__ void embed_rows_kernel(const TT* __restrict__ table, const int* __restrict__ ids,
                                  float* __restrict__ out, int hidden, int vocab, int copies, long long copy_stride) {
  pdl_launch_dependents();
  pdl_wait();
  const int n = blockIdx.x;
  int id = ids[n];
  if (id < 0 || id >= vocab) id = 0;  // ids are validated on the host; never read out of range
  const TT* row = table + (long long)id * hidden;
  float* o = out + (long long)n * hidden;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    const float v = to_f32(row[i]);
    for (int c = 0; c < copies; ++c) o[c * copy_stride + i] = v;
  }
}

// residual[n][:] = table[ids[n]][:]   (no scaling; Inference/ForwardPass.cs:205)
// With copies > 1 the row is written `copies` times, `copy_stride` elements apart (a residual of several streams that all
// start as the embedding: out is [copies][n_tokens][hidden]).
LLG_API int llg_embed_rows_copies(const void* table, int table_dtype, const int* ids, float* out, int n_tokens, int hidden,
                                  int vocab, int copies, long long copy_stride, cudaStream_t stream) {
  LLG_REQUIRE(n_tokens >= 0 && hidden > 0 && vocab > 0 && copies >= 1, "embed_rows: bad sizes n=%d hidden=%d vocab=%d copies=%d",
              n_tokens, hidden, vocab, copies);
  if (n_tokens == 0) return 0;
  const int threads = hidden >= 1024 ? 256 : 128;
  if (table_dtype == LLG_F32)
    llg_launch(embed_rows_kernel<float>, n_tokens, threads, 0, stream, (const float*)table, ids, out, hidden, vocab, copies, copy_stride);
  else if (table_dtype == LLG_BF16)
    llg_launch(embed_rows_kernel<__nv_bfloat16>, n_tokens, threads, 0, stream, (const __nv_bfloat16*)table, ids, out, hidden, vocab,
               copies, copy_stride);
  else
    return llg_fail("embed_rows: unknown table dtype %d", table_dtype);
  return llg_check_launch("embed_rows");
}

LLG_API int llg_embed_rows(const void* table, int table_dtype, const int* ids, float* out,
                           int n_tokens, int hidden, int vocab, cudaStream_t stream) {
  return llg_embed_rows_copies(table, table_dtype, ids, out, n_tokens, hidden, vocab, 1, 0, stream);
}

// four consecutive elements as float32 (the address is a multiple of 4 elements)
__device__ __forceinline__ void vec_load4(const float* p, float (&v)[4]) {
  const float4 t = *reinterpret_cast<const float4*>(p);
  v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
}
__device__ __forceinline__ void vec_load4(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 t = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&t.x), hi = *reinterpret_cast<const __nv_bfloat162*>(&t.y);
  v[0] = __low2float(lo); v[1] = __high2float(lo); v[2] = __low2float(hi); v[3] = __high2float(hi);
}
__device__ __forceinline__ void vec_store4(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void vec_store4(__nv_bfloat16* p, const float (&v)[4]) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
  uint2 t;
  t.x = *reinterpret_cast<const uint32_t*>(&lo);
  t.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = t;
}

// ---- residual add + RMSNorm ---------------------------------------------------------

// For output row j (token r = rows ? rows[j] : j):
//   v = residual[r] + branch_bias + sum_s branch[s][r]   (written back to residual when there is a branch)
//   out[j] = v * rsqrt(mean(v^2) + eps) * weight         (eps inside the root, weight after)
// With ss_out the division is left to the consumer of out (RowScale in kernel_args.h): out[j] = v * weight and
// ss_out[j] = sum(v^2), whole or in parts.
template <typename OT, typename WT>
__global__ void add_rmsnorm_kernel(float* __restrict__ residual, const float* __restrict__ branch,
                                   int n_partials, long long partial_stride, const WT* __restrict__ weight,
                                   float eps, OT* __restrict__ out, const int* __restrict__ rows, int hidden,
                                   float* __restrict__ ss_out, const float* __restrict__ branch_bias) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const int j = blockIdx.x;
  const int r = rows ? rows[j] : j;
  float* res = residual + (long long)r * hidden;
  float ss = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    float v = res[i];
    if (branch) {
      const float* b = branch + (long long)r * hidden + i;
      if (branch_bias) v += branch_bias[i];
      for (int s = 0; s < n_partials; ++s) v += b[s * partial_stride];
      res[i] = v;
    }
    ss += v * v;
  }
  ss = block_sum(ss, red);
  const float inv = ss_out ? 1.0f : 1.0f / sqrtf(ss / (float)hidden + eps);
  if (ss_out && threadIdx.x == 0) ss_out[j] = ss;
  OT* o = out + (long long)j * hidden;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x)
    o[i] = from_f32<OT>(res[i] * inv * to_f32(weight[i]));
}

// The same for rows whose length is a multiple of 4: 16-byte accesses, the row stays in registers
// between the two passes (VPT float4 per thread), and the partials of one element are loaded together
// so that their latencies overlap (a decode step has few rows and nothing else to hide them behind).
// One block per row also for the few rows of a decode step: a row spread over a cluster of eight blocks
// (sums of squares exchanged through distributed shared memory) took 0.07 ms more per step of 32 layers.
template <typename OT, typename WT, int VPT>
__global__ void add_rmsnorm_vec4_kernel(float* __restrict__ residual, const float* __restrict__ branch,
                                        int n_partials, long long partial_stride, const WT* __restrict__ weight,
                                        float eps, OT* __restrict__ out, const int* __restrict__ rows, int hidden,
                                        float* __restrict__ ss_out, const float* __restrict__ branch_bias) {
  __shared__ float red[32];
  pdl_launch_dependents();
  const int nv = hidden >> 2;
  // the norm's weight is no result of an earlier kernel: fetch it while the predecessor still runs
  float wv[VPT][4];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < nv) vec_load4(weight + 4 * i, wv[k]);
  }
  if (threadIdx.x == 0) LLG_STAMP(3, 0, 0, blockIdx.x);
  pdl_wait();
  if (threadIdx.x == 0) LLG_STAMP(3, 1, 0, blockIdx.x);
  const int j = blockIdx.x;
  const int r = rows ? rows[j] : j;
  float4* res = reinterpret_cast<float4*>(residual + (long long)r * hidden);
  float4 keep[VPT];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < nv) {
      v = res[i];
      if (branch) {
        if (branch_bias) {
          const float4 bb = reinterpret_cast<const float4*>(branch_bias)[i];
          v.x += bb.x; v.y += bb.y; v.z += bb.z; v.w += bb.w;
        }
        const float4* b = reinterpret_cast<const float4*>(branch + (long long)r * hidden) + i;
        const long long ps = partial_stride >> 2;
        int s = 0;
        if (VPT == 1) {
          // few rows (one float4 a thread): nothing to hide a load behind, so the first twelve partials are all asked
          // for before the first is added (one trip to L2 instead of one per group); they are added in their order
          constexpr int AT_ONCE = 12;
          float4 pv[AT_ONCE];
#pragma unroll
          for (int q = 0; q < AT_ONCE; ++q) pv[q] = q < n_partials ? b[q * ps] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
          for (int q = 0; q < AT_ONCE; ++q)
            if (q < n_partials) { v.x += pv[q].x; v.y += pv[q].y; v.z += pv[q].z; v.w += pv[q].w; }
          s = n_partials < AT_ONCE ? n_partials : AT_ONCE;
        }
        for (; s + 4 <= n_partials; s += 4) {
          const float4 b0 = b[(s + 0) * ps], b1 = b[(s + 1) * ps], b2 = b[(s + 2) * ps], b3 = b[(s + 3) * ps];
          v.x += b0.x; v.y += b0.y; v.z += b0.z; v.w += b0.w;
          v.x += b1.x; v.y += b1.y; v.z += b1.z; v.w += b1.w;
          v.x += b2.x; v.y += b2.y; v.z += b2.z; v.w += b2.w;
          v.x += b3.x; v.y += b3.y; v.z += b3.z; v.w += b3.w;
        }
        for (; s < n_partials; ++s) {
          const float4 b0 = b[s * ps];
          v.x += b0.x; v.y += b0.y; v.z += b0.z; v.w += b0.w;
        }
        res[i] = v;
      }
    }
    keep[k] = v;
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  ss = block_sum(ss, red);
  const float inv = ss_out ? 1.0f : 1.0f / sqrtf(ss / (float)hidden + eps);
  if (ss_out && threadIdx.x == 0) ss_out[j] = ss;
  OT* o = out + (long long)j * hidden;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < nv) {
      const float4 v = keep[k];
      const float y[4] = {v.x * inv * wv[k][0], v.y * inv * wv[k][1], v.z * inv * wv[k][2], v.w * inv * wv[k][3]};
      vec_store4(o + 4 * i, y);
    }
  }
  if (threadIdx.x == 0) LLG_STAMP(3, 3, 0, blockIdx.x);
}

// The norm of a step of few rows when the division is left to the consumer: nothing then needs a whole row, so a
// row is cut into slices of PARTS_THREADS float4 and every (slice, row) is a block of its own that adds up its
// columns' partial sums, writes the residual stream, the weighted row and its slice's sum of squares (the consumer
// adds the slices' sums in their order).  One multiprocessor fetches a row's partial sums at some 40 GB/s (4 us
// for the 147 KB of a 4096-wide row with nine partials); spread over sixteen blocks they are there in one trip.
constexpr int PARTS_THREADS = 64;

template <typename OT, typename WT>
__global__ void __launch_bounds__(PARTS_THREADS) add_rmsnorm_parts_kernel(float* __restrict__ residual, const float* __restrict__ branch,
                                                                           int n_partials, long long partial_stride,
                                                                           const WT* __restrict__ weight, OT* __restrict__ out,
                                                                           const int* __restrict__ rows, int hidden,
                                                                           float* __restrict__ ss_out,
                                                                           const float* __restrict__ branch_bias) {
  __shared__ float red[32];
  pdl_launch_dependents();
  const int i = blockIdx.x * PARTS_THREADS + threadIdx.x;          // float4 of the row (the host checks divisibility)
  float wv[4];
  vec_load4(weight + 4 * i, wv);                                   // no result of an earlier kernel
  float4 bb = make_float4(0.f, 0.f, 0.f, 0.f);
  if (branch_bias) bb = reinterpret_cast<const float4*>(branch_bias)[i];
  const int j = blockIdx.y;
  if (threadIdx.x == 0) LLG_STAMP(3, 0, 0, blockIdx.x + gridDim.x * blockIdx.y);
  pdl_wait();
  if (threadIdx.x == 0) LLG_STAMP(3, 1, 0, blockIdx.x + gridDim.x * blockIdx.y);
  const int r = rows ? rows[j] : j;
  float4* res = reinterpret_cast<float4*>(residual + (long long)r * hidden);
  float4 v = res[i];
  if (branch) {
    if (branch_bias) { v.x += bb.x; v.y += bb.y; v.z += bb.z; v.w += bb.w; }
    const float4* b = reinterpret_cast<const float4*>(branch + (long long)r * hidden) + i;
    const long long ps = partial_stride >> 2;
    constexpr int AT_ONCE = 12;                                    // all asked for before the first is added, added in order
    float4 pv[AT_ONCE];
#pragma unroll
    for (int q = 0; q < AT_ONCE; ++q) pv[q] = q < n_partials ? b[q * ps] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int q = 0; q < AT_ONCE; ++q)
      if (q < n_partials) { v.x += pv[q].x; v.y += pv[q].y; v.z += pv[q].z; v.w += pv[q].w; }
    for (int q = AT_ONCE; q < n_partials; ++q) {
      const float4 b0 = b[q * ps];
      v.x += b0.x; v.y += b0.y; v.z += b0.z; v.w += b0.w;
    }
    res[i] = v;
  }
  const float y[4] = {v.x * wv[0], v.y * wv[1], v.z * wv[2], v.w * wv[3]};
  vec_store4(out + (long long)j * hidden + 4 * i, y);
  const float ss = block_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w, red);
  if (threadIdx.x == 0) ss_out[(long long)j * gridDim.x + blockIdx.x] = ss;
  if (threadIdx.x == 0) LLG_STAMP(3, 3, 0, blockIdx.x + gridDim.x * blockIdx.y);
}

// Parts that llg_add_rmsnorm writes per row into ss_out for these sizes (the consumer's RowScale.parts).
LLG_API int llg_add_rmsnorm_parts(int n_out, int hidden) {
  const bool spread = n_out <= 64 && hidden >= 1024 && hidden % (4 * PARTS_THREADS) == 0 && hidden / (4 * PARTS_THREADS) <= 64;
  return spread ? hidden / (4 * PARTS_THREADS) : 1;
}

LLG_API int llg_add_rmsnorm(float* residual, const float* branch, int n_partials, long long partial_stride,
                            const void* weight, int weight_dtype, float eps, void* out, int out_dtype,
                            const int* rows, int n_out, int hidden, float* ss_out, const float* branch_bias, cudaStream_t stream) {
  LLG_REQUIRE(n_out >= 0 && hidden > 0, "add_rmsnorm: bad sizes n_out=%d hidden=%d", n_out, hidden);
  LLG_REQUIRE(eps > 0.f, "add_rmsnorm: eps must be positive");
  LLG_REQUIRE(!branch || n_partials >= 1, "add_rmsnorm: a branch needs n_partials >= 1");
  LLG_REQUIRE(branch || !branch_bias, "add_rmsnorm: a bias without a branch");
  if (n_out == 0) return 0;
  const bool vec = hidden % 4 == 0 && partial_stride % 4 == 0 && ((uintptr_t)residual % 16) == 0 &&
                   ((uintptr_t)branch % 16) == 0 && ((uintptr_t)weight % 16) == 0 && ((uintptr_t)out % 16) == 0 &&
                   ((uintptr_t)branch_bias % 16) == 0;
  int threads = hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128);
  // vector path: few rows (decode) want many threads per row, many rows want the row in registers
  int vpt = 1;
  if (vec) {
    const int nv = hidden / 4;
    if (n_out <= 256) {
      threads = nv >= 1024 ? 1024 : (nv >= 256 ? 256 : 128);
    } else {
      threads = nv >= 1024 ? 512 : 256;
    }
    vpt = (nv + threads - 1) / threads;
    if (vpt > 8) {                     // rows longer than 8 float4 per thread: more threads
      threads = 1024;
      vpt = (nv + threads - 1) / threads;
    }
  }
  const bool vec_ok = vec && vpt <= 8;
  // the division left to the consumer and few rows: every slice of a row is a block of its own
  const int parts = ss_out ? llg_add_rmsnorm_parts(n_out, hidden) : 1;
  LLG_REQUIRE(parts == 1 || vec, "add_rmsnorm: operands of a norm in parts must be 16-byte aligned");
#define LAUNCH(OT, WT)                                                                                         \
  do {                                                                                                         \
    if (parts > 1)                                                                                             \
      llg_launch(add_rmsnorm_parts_kernel<OT, WT>, dim3(parts, n_out), PARTS_THREADS, 0, stream, residual, branch, \
                 n_partials, partial_stride, (const WT*)weight, (OT*)out, rows, hidden, ss_out, branch_bias);               \
    else if (vec_ok && vpt <= 1)                                                                                    \
      llg_launch(add_rmsnorm_vec4_kernel<OT, WT, 1>, n_out, threads, 0, stream, residual, branch, n_partials,    \
                 partial_stride, (const WT*)weight, eps, (OT*)out, rows, hidden, ss_out, branch_bias);                      \
    else if (vec_ok && vpt <= 2)                                                                               \
      llg_launch(add_rmsnorm_vec4_kernel<OT, WT, 2>, n_out, threads, 0, stream, residual, branch, n_partials,    \
                 partial_stride, (const WT*)weight, eps, (OT*)out, rows, hidden, ss_out, branch_bias);                      \
    else if (vec_ok && vpt <= 4)                                                                               \
      llg_launch(add_rmsnorm_vec4_kernel<OT, WT, 4>, n_out, threads, 0, stream, residual, branch, n_partials,    \
                 partial_stride, (const WT*)weight, eps, (OT*)out, rows, hidden, ss_out, branch_bias);                      \
    else if (vec_ok)                                                                                           \
      llg_launch(add_rmsnorm_vec4_kernel<OT, WT, 8>, n_out, threads, 0, stream, residual, branch, n_partials,    \
                 partial_stride, (const WT*)weight, eps, (OT*)out, rows, hidden, ss_out, branch_bias);                      \
    else                                                                                                       \
      llg_launch(add_rmsnorm_kernel<OT, WT>, n_out, threads, 0, stream, residual, branch, n_partials,            \
                 partial_stride, (const WT*)weight, eps, (OT*)out, rows, hidden, ss_out, branch_bias);                      \
  } while (0)
  if (out_dtype == LLG_F32 && weight_dtype == LLG_F32) LAUNCH(float, float);
  else if (out_dtype == LLG_F32 && weight_dtype == LLG_BF16) LAUNCH(float, __nv_bfloat16);
  else if (out_dtype == LLG_BF16 && weight_dtype == LLG_F32) LAUNCH(__nv_bfloat16, float);
  else if (out_dtype == LLG_BF16 && weight_dtype == LLG_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else return llg_fail("add_rmsnorm: unknown dtypes out=%d weight=%d", out_dtype, weight_dtype);
#undef LAUNCH
  return llg_check_launch("add_rmsnorm");
}

// ---- query/key preparation ----------------------------------------------------------

// What queries at a position are multiplied by (QkPrepArgs.q_scale; the host checks the table's reach).
__device__ __forceinline__ float query_scale(const QkPrepArgs& a, int pos) {
  return a.q_scale ? a.q_scale[pos < a.q_scale_positions ? pos : a.q_scale_positions - 1] : 1.0f;
}

template <typename IT, typename OT, typename WT>
__global__ void qk_prep_kernel(QkPrepArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float sm[];
  const int warps = blockDim.x >> 5;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int heads = a.nh + 2 * a.nkv, units = heads + (a.gate_out ? 1 : 0);     // the gates of a token's heads are one unit more
  const long long item = (long long)blockIdx.x * warps + warp;
  if (item >= (long long)a.n_tokens * units) return;
  const int n = (int)(item / units);
  const int h = (int)(item % units);
  const int kind = h < a.nh ? 0 : (h < a.nh + a.nkv ? 1 : 2);  // 0 query, 1 key, 2 value
  const int vd = a.vd > 0 ? a.vd : a.hd;
  const int hd = kind == 2 ? vd : a.hd;                        // elements of this head
  float* x = sm + warp * max(a.hd, vd);
  const long long qkv_w = (long long)(a.nh + a.nkv) * a.hd + (long long)a.nkv * vd;
  const long long row_w = qkv_w + (a.gate_out ? a.nh : 0);
  if (h == heads) {
    const IT* z = (const IT*)a.qkv + (long long)n * row_w + qkv_w;
    const float zs = row_scale_of(a.row_scale, n);
    for (int i = lane; i < a.nh; i += 32) {
      float v = 0.f;
      for (int s = 0; s < a.n_partials; ++s) v += to_f32(z[s * a.partial_stride + i]);
      a.gate_out[(long long)n * a.nh + i] = 1.0f / (1.0f + expf(-v * zs));
    }
    return;
  }
  const long long col = kind == 2 ? (long long)(a.nh + a.nkv) * a.hd + (long long)(h - a.nh - a.nkv) * vd : (long long)h * a.hd;
  const long long off = (long long)n * row_w + col;
  const IT* src = (const IT*)a.qkv + off;

  const float rs = row_scale_of(a.row_scale, n);
  float ss = 0.f;
  for (int d = lane; d < hd; d += 32) {
    float v = 0.f;
    for (int s = 0; s < a.n_partials; ++s) v += to_f32(src[s * a.partial_stride + d]);
    v *= rs;
    x[d] = v;
    ss += v * v;
  }
  const WT* nw = kind == 0 ? (const WT*)a.q_norm_w : (kind == 1 ? (const WT*)a.k_norm_w : nullptr);
  if (nw) {  // per-head RMSNorm first, then bias, then rotation (Inference/ForwardPass.cs:372-385)
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)hd + a.norm_eps);
    for (int d = lane; d < hd; d += 32) x[d] = x[d] * inv * to_f32(nw[d]);
  }
  if (a.bias) {
    const WT* b = (const WT*)a.bias + col;
    for (int d = lane; d < hd; d += 32) x[d] += to_f32(b[d]);
  }
  if (kind == 2 && (a.v_first_out || a.v_first_in)) {
    // values blended across layers: the first layer of a group lends its values as projected, the others keep
    // (1 - lam) v + lam v_first; all of it in float32
    const long long vo = ((long long)n * a.nkv + (h - a.nh - a.nkv)) * vd;
    if (a.v_first_out)
      for (int d = lane; d < hd; d += 32) a.v_first_out[vo + d] = x[d];
    if (a.v_first_in) {
      const float lam = a.v_mix[0];
      for (int d = lane; d < hd; d += 32) x[d] = (1.0f - lam) * x[d] + lam * a.v_first_in[vo + d];
    }
  }
  __syncwarp();
  const int pos = a.positions[n];
  if (kind != 2 && a.cos_table) {
    const int half = a.rotary_dim >> 1;
    const int p = pos < a.table_positions ? pos : a.table_positions - 1;  // bounded; host checks capacity
    const float* c = a.cos_table + (long long)p * half;
    const float* s = a.sin_table + (long long)p * half;
    for (int i = lane; i < half; i += 32) {
      const int i0 = a.pairing == 0 ? i : 2 * i;
      const int i1 = a.pairing == 0 ? i + half : 2 * i + 1;
      const float x0 = x[i0], x1 = x[i1];
      const float cs = c[i], sn = s[i];
      x[i0] = x0 * cs - x1 * sn;
      x[i1] = x0 * sn + x1 * cs;
    }
    __syncwarp();
  }
  if (kind == 0) {
    const float qs = query_scale(a, pos);
    if (a.q_maps == 2) {
      OT* o = (OT*)a.q_out + ((long long)n * a.nh + h) * 2 * hd;
      for (int d = lane; d < hd; d += 32) {
        const float v = x[d] * qs;
        o[d] = from_f32<OT>(2 * d < hd ? v : 0.f);
        o[hd + d] = from_f32<OT>(2 * d < hd ? 0.f : v);
      }
      return;
    }
    OT* o = (OT*)a.q_out + ((long long)n * a.nh + h) * hd;
    for (int d = lane; d < hd; d += 32) o[d] = from_f32<OT>(x[d] * qs);
    return;
  }
  const int kvh = kind == 1 ? h - a.nh : h - a.nh - a.nkv;
  void* packed = kind == 1 ? a.k_new : a.v_new;
  if (packed) {
    OT* o = (OT*)packed + ((long long)n * a.nkv + kvh) * hd;
    for (int d = lane; d < hd; d += 32) o[d] = from_f32<OT>(x[d]);
  }
  void* pages = kind == 1 ? a.k_pages : a.v_pages;
  if (pages) {
    const int slot = a.slots[a.seq_of_token[n]];
    const long long row = kv_row(a.page_table, a.table_width, a.ring_pages, slot, pos, kvh, a.nkv);
    OT* o = (OT*)pages + row * hd;
    for (int d = lane; d < hd; d += 32) o[d] = from_f32<OT>(x[d]);
  }
}

// The same for the common geometry (head size 64, 128 or 256; rotation by halves over the whole
// head, or none): HD / 8 lanes share a head; a lane keeps elements 4l .. 4l+3 of each half in
// registers, so a rotation pair (i, i + HD / 2) lies in one lane, every access moves four elements,
// nothing goes through shared memory, and all loads of a head are issued before the first use.
template <typename IT, typename OT, typename WT, int HD>
__global__ void __launch_bounds__(256) qk_prep_vec_kernel(QkPrepArgs a) {
  pdl_launch_dependents();
  constexpr int LPH = HD / 8, HALF = HD / 2;      // lanes per head
  const int heads = a.nh + 2 * a.nkv;
  const long long item = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / LPH;
  const int l = threadIdx.x % LPH;
  // lanes past the last head still take part in the shuffles below
  const bool live = item < (long long)a.n_tokens * heads;
  const int n = live ? (int)(item / heads) : 0;
  const int h = live ? (int)(item % heads) : 0;
  const int kind = h < a.nh ? 0 : (h < a.nh + a.nkv ? 1 : 2);
  const int kvh = kind == 1 ? h - a.nh : h - a.nh - a.nkv;
  // Everything but the sums themselves was written before this step's first kernel started (positions, the batch's
  // slots, the page table) or never changes (weights, biases, rotation tables): it is fetched while the product ahead
  // still runs, so that after the wait only the sums are a trip to memory away.
  const WT* nw = kind == 0 ? (const WT*)a.q_norm_w : (kind == 1 ? (const WT*)a.k_norm_w : nullptr);
  float w0[4] = {1.f, 1.f, 1.f, 1.f}, w1[4] = {1.f, 1.f, 1.f, 1.f}, b0[4] = {0.f, 0.f, 0.f, 0.f}, b1[4] = {0.f, 0.f, 0.f, 0.f};
  float cs[4] = {1.f, 1.f, 1.f, 1.f}, si[4] = {0.f, 0.f, 0.f, 0.f};
  if (nw) {
    vec_load4(nw + 4 * l, w0);
    vec_load4(nw + 4 * l + HALF, w1);
  }
  if (a.bias && live) {
    const WT* bsrc = (const WT*)a.bias + (long long)h * HD + 4 * l;
    vec_load4(bsrc, b0);
    vec_load4(bsrc + HALF, b1);
  }
  const int pos = a.positions[n];
  const float qs = kind == 0 ? query_scale(a, pos) : 1.0f;
  const bool rotate = kind != 2 && a.cos_table;
  if (rotate) {
    const int p = pos < a.table_positions ? pos : a.table_positions - 1;
    vec_load4(a.cos_table + (long long)p * HALF + 4 * l, cs);
    vec_load4(a.sin_table + (long long)p * HALF + 4 * l, si);
  }
  void* pages = kind == 0 ? nullptr : (kind == 1 ? a.k_pages : a.v_pages);
  long long page_row = 0;
  if (pages && live) page_row = kv_row(a.page_table, a.table_width, a.ring_pages, a.slots[a.seq_of_token[n]], pos, kvh, a.nkv);
  if (threadIdx.x == 0) LLG_STAMP(4, 0, 0, blockIdx.x);
  pdl_wait();
  if (threadIdx.x == 0) LLG_STAMP(4, 1, 0, blockIdx.x);
  const float rs = row_scale_of(a.row_scale, n);      // the norm's sums: a kernel of this step wrote them, so after the wait
  const IT* src = (const IT*)a.qkv + (long long)n * heads * HD + (long long)h * HD + 4 * l;
  float x0[4] = {0.f, 0.f, 0.f, 0.f}, x1[4] = {0.f, 0.f, 0.f, 0.f};   // elements 4l.. of the first and second half
  // the first eight partials are all asked for before the first is added; they are added in their order
  constexpr int AT_ONCE = 8;
  float t0[AT_ONCE][4], t1[AT_ONCE][4];
#pragma unroll
  for (int s = 0; s < AT_ONCE; ++s) {
    if (s < a.n_partials) {
      vec_load4(src + s * a.partial_stride, t0[s]);
      vec_load4(src + s * a.partial_stride + HALF, t1[s]);
    }
  }
#pragma unroll
  for (int s = 0; s < AT_ONCE; ++s) {
    if (s < a.n_partials) {
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        x0[k] += t0[s][k];
        x1[k] += t1[s][k];
      }
    }
  }
  for (int s = AT_ONCE; s < a.n_partials; ++s) {
    float u0[4], u1[4];
    vec_load4(src + s * a.partial_stride, u0);
    vec_load4(src + s * a.partial_stride + HALF, u1);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      x0[k] += u0[k];
      x1[k] += u1[k];
    }
  }
  if (a.row_scale.ss) {                             // what the norm ahead left to its consumer
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      x0[k] *= rs;
      x1[k] *= rs;
    }
  }
  if (a.q_norm_w || a.k_norm_w) {                  // uniform over the block: the shuffles need every lane
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) ss += x0[k] * x0[k] + x1[k] * x1[k];
#pragma unroll
    for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (nw) {
      const float inv = 1.0f / sqrtf(ss / (float)HD + a.norm_eps);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        x0[k] = x0[k] * inv * w0[k];
        x1[k] = x1[k] * inv * w1[k];
      }
    }
  }
  if (!live) return;
  if (a.bias) {
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      x0[k] += b0[k];
      x1[k] += b1[k];
    }
  }
  if (rotate) {
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float u = x0[k], v = x1[k];
      x0[k] = u * cs[k] - v * si[k];
      x1[k] = u * si[k] + v * cs[k];
    }
  }
  if (kind == 0) {
    if (a.q_scale) {
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        x0[k] *= qs;
        x1[k] *= qs;
      }
    }
    if (a.q_maps == 2) {
      const float none[4] = {0.f, 0.f, 0.f, 0.f};
      OT* o = (OT*)a.q_out + ((long long)n * a.nh + h) * 2 * HD + 4 * l;
      vec_store4(o, x0);
      vec_store4(o + HALF, none);
      vec_store4(o + HD, none);
      vec_store4(o + HD + HALF, x1);
      return;
    }
    OT* o = (OT*)a.q_out + ((long long)n * a.nh + h) * HD + 4 * l;
    vec_store4(o, x0);
    vec_store4(o + HALF, x1);
    return;
  }
  void* packed = kind == 1 ? a.k_new : a.v_new;
  if (packed) {
    OT* o = (OT*)packed + ((long long)n * a.nkv + kvh) * HD + 4 * l;
    vec_store4(o, x0);
    vec_store4(o + HALF, x1);
  }
  if (pages) {
    OT* o = (OT*)pages + page_row * HD + 4 * l;
    vec_store4(o, x0);
    vec_store4(o + HALF, x1);
  }
  if (threadIdx.x == 0) LLG_STAMP(4, 3, 0, blockIdx.x);
}

LLG_API int llg_qk_prep(const QkPrepArgs* args, int out_dtype, cudaStream_t stream) {
  const QkPrepArgs& a = *args;
  LLG_REQUIRE(a.n_tokens >= 0 && a.nh > 0 && a.nkv >= 0 && a.hd > 0, "qk_prep: bad sizes");
  LLG_REQUIRE(a.hd <= 1024, "qk_prep: head_dim %d is larger than 1024", a.hd);
  LLG_REQUIRE(!a.cos_table || (a.rotary_dim > 0 && a.rotary_dim % 2 == 0 && a.rotary_dim <= a.hd),
              "qk_prep: rotary_dim %d must be even and at most head_dim %d", a.rotary_dim, a.hd);
  LLG_REQUIRE(a.n_partials >= 1, "qk_prep: n_partials must be >= 1");
  LLG_REQUIRE(a.q_maps == 0 || (a.q_maps == 2 && a.hd % 2 == 0), "qk_prep: %d maps of a query of %d elements (0 or 2)", a.q_maps, a.hd);
  LLG_REQUIRE(!a.q_scale || a.q_scale_positions > 0, "qk_prep: an empty table of query factors");
  LLG_REQUIRE(!a.k_pages || (a.page_table && a.slots && a.seq_of_token && a.ring_pages > 0),
              "qk_prep: a cache write needs page_table, slots and seq_of_token");
  if (a.n_tokens == 0) return 0;
  // the vector kernel moves four elements at a time: every pointer must be 16-byte aligned
  auto aligned = [](const void* p) { return ((uintptr_t)p & 15u) == 0; };
  const bool plain_values = (a.vd == 0 || a.vd == a.hd) && !a.v_first_in && !a.v_first_out;
  LLG_REQUIRE(a.vd >= 0 && a.vd <= 1024, "qk_prep: value head size %d is larger than 1024", a.vd);
  LLG_REQUIRE(!a.v_first_in || a.v_mix, "qk_prep: blending values needs the blend's weight");
  const bool lane_ok = plain_values && !a.gate_out && (a.hd == 64 || a.hd == 128 || a.hd == 256) &&
                       (!a.cos_table || (a.pairing == 0 && a.rotary_dim == a.hd)) && a.partial_stride % 4 == 0 &&
                       aligned(a.qkv) && aligned(a.q_norm_w) && aligned(a.k_norm_w) && aligned(a.bias) &&
                       aligned(a.cos_table) && aligned(a.sin_table) && aligned(a.q_out) && aligned(a.k_new) &&
                       aligned(a.v_new) && aligned(a.k_pages) && aligned(a.v_pages);
  const long long items = (long long)a.n_tokens * (a.nh + 2 * a.nkv + (a.gate_out ? 1 : 0));
  // a step of few tokens spreads its heads over many small blocks: nothing but memory latency bounds it
  const bool few = lane_ok && items * (a.hd / 8) <= (long long)2 * 64 * llg_sm_count();
  const int warps = lane_ok ? (few ? 2 : 8) : 4;
  // the vector kernel gives a head to head_dim / 8 lanes, the general one to a warp
  const long long per_block = lane_ok ? (long long)warps * 32 / (a.hd / 8) : warps;
  const unsigned grid = (unsigned)((items + per_block - 1) / per_block);
  const size_t smem = lane_ok ? 0 : (size_t)warps * (a.hd > a.vd ? a.hd : a.vd) * sizeof(float);
  const bool w_bf16 = (a.q_norm_w || a.k_norm_w) ? a.norm_w_dtype == LLG_BF16
                                                 : (a.bias ? a.bias_dtype == LLG_BF16 : false);
  if ((a.q_norm_w || a.k_norm_w) && a.bias)
    LLG_REQUIRE(a.norm_w_dtype == a.bias_dtype, "qk_prep: norm weights and bias must share a dtype");
#define LAUNCH(IT, OT, WT)                                                        \
  do {                                                                            \
    if (lane_ok && a.hd == 64) llg_launch(qk_prep_vec_kernel<IT, OT, WT, 64>, grid, warps * 32, 0, stream, a);        \
    else if (lane_ok && a.hd == 128) llg_launch(qk_prep_vec_kernel<IT, OT, WT, 128>, grid, warps * 32, 0, stream, a);  \
    else if (lane_ok) llg_launch(qk_prep_vec_kernel<IT, OT, WT, 256>, grid, warps * 32, 0, stream, a);                 \
    else llg_launch(qk_prep_kernel<IT, OT, WT>, grid, warps * 32, smem, stream, a);         \
  } while (0)
  if (out_dtype == LLG_F32) {
    LLG_REQUIRE(a.qkv_dtype == LLG_F32, "qk_prep: float32 output needs float32 input");
    if (w_bf16) LAUNCH(float, float, __nv_bfloat16); else LAUNCH(float, float, float);
  } else if (out_dtype == LLG_BF16) {
    if (a.qkv_dtype == LLG_F32) {
      if (w_bf16) LAUNCH(float, __nv_bfloat16, __nv_bfloat16); else LAUNCH(float, __nv_bfloat16, float);
    } else {
      if (w_bf16) LAUNCH(__nv_bfloat16, __nv_bfloat16, __nv_bfloat16);
      else LAUNCH(__nv_bfloat16, __nv_bfloat16, float);
    }
  } else {
    return llg_fail("qk_prep: unknown output dtype %d", out_dtype);
  }
#undef LAUNCH
  return llg_check_launch("qk_prep");
}

// ---- the difference of two maps' outputs -------------------------------------------
//
// raw [n_tokens][nh][2][vd] float32: o = raw[.][0] - lambda raw[.][1], divided by sqrt(mean(o^2) + eps) over the vd elements of a
// head and multiplied by scale.  A warp per (token, head).
template <typename OT>
__global__ void __launch_bounds__(128) map_difference_kernel(const float* __restrict__ raw, OT* __restrict__ out, long long items, int vd,
                                                             float lambda, float eps, float scale) {
  pdl_launch_dependents();
  pdl_wait();
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= items) return;
  const float *r1 = raw + item * 2 * vd, *r2 = r1 + vd;
  OT* o = out + item * vd;
  float ss = 0.f;
  if ((vd & 3) == 0 && vd <= 512) {
    float v[4][4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int d = 4 * (lane + 32 * k);
      if (d < vd) {
        float a1[4], a2[4];
        vec_load4(r1 + d, a1);
        vec_load4(r2 + d, a2);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          v[k][e] = fmaf(-lambda, a2[e], a1[e]);
          ss = fmaf(v[k][e], v[k][e], ss);
        }
      }
    }
    const float f = scale / sqrtf(warp_sum(ss) / (float)vd + eps);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int d = 4 * (lane + 32 * k);
      if (d < vd) {
        const float y[4] = {v[k][0] * f, v[k][1] * f, v[k][2] * f, v[k][3] * f};
        vec_store4(o + d, y);
      }
    }
    return;
  }
  for (int d = lane; d < vd; d += 32) {
    const float v = fmaf(-lambda, r2[d], r1[d]);
    ss = fmaf(v, v, ss);
  }
  const float f = scale / sqrtf(warp_sum(ss) / (float)vd + eps);
  for (int d = lane; d < vd; d += 32) o[d] = from_f32<OT>(fmaf(-lambda, r2[d], r1[d]) * f);
}

LLG_API int llg_map_difference(const float* raw, void* out, int out_dtype, int n_tokens, int nh, int vd, float lambda, float eps,
                               float scale, cudaStream_t stream) {
  LLG_REQUIRE(n_tokens >= 0 && nh > 0 && vd > 0 && eps > 0.f, "map_difference: bad sizes");
  LLG_REQUIRE(((uintptr_t)raw & 15u) == 0 && ((uintptr_t)out & 15u) == 0, "map_difference: operands must be 16-byte aligned");
  if (n_tokens == 0) return 0;
  const long long items = (long long)n_tokens * nh;
  const unsigned grid = (unsigned)((items + 3) / 4);
  if (out_dtype == LLG_F32) llg_launch(map_difference_kernel<float>, grid, 128, 0, stream, raw, (float*)out, items, vd, lambda, eps, scale);
  else if (out_dtype == LLG_BF16)
    llg_launch(map_difference_kernel<__nv_bfloat16>, grid, 128, 0, stream, raw, (__nv_bfloat16*)out, items, vd, lambda, eps, scale);
  else return llg_fail("map_difference: unknown output type %d", out_dtype);
  return llg_check_launch("map_difference");
}

// ---- cache write after a prompt step ------------------------------------------------

// Copies this step's keys and values [n_tokens][nkv][hd] into the paged store.  A token whose
// ring position would be overwritten by a later token of the same step is skipped.
template <typename T>
__global__ void kv_write_kernel(const T* __restrict__ k_new, const T* __restrict__ v_new, T* __restrict__ k_pages,
                                T* __restrict__ v_pages, const int* __restrict__ page_table, int table_width,
                                int ring_pages, const int* __restrict__ positions,
                                const int* __restrict__ seq_of_token, const int* __restrict__ slots,
                                const int* __restrict__ cu_tokens, const int* __restrict__ len_before,
                                int n_tokens, int nkv, int hd) {
  pdl_launch_dependents();
  pdl_wait();
  const int warps = blockDim.x >> 5;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * warps + warp;
  if (item >= (long long)n_tokens * nkv) return;
  const int n = (int)(item / nkv), kvh = (int)(item % nkv);
  const int b = seq_of_token[n];
  const int pos = positions[n];
  const int len_after = len_before[b] + (cu_tokens[b + 1] - cu_tokens[b]);
  if (pos < len_after - ring_pages * LLG_PAGE) return;
  const long long row = kv_row(page_table, table_width, ring_pages, slots[b], pos, kvh, nkv);
  const T* ks = k_new + ((long long)n * nkv + kvh) * hd;
  const T* vs = v_new + ((long long)n * nkv + kvh) * hd;
  T* kd = k_pages + row * hd;
  T* vd = v_pages + row * hd;
  for (int d = lane; d < hd; d += 32) {
    kd[d] = ks[d];
    vd[d] = vs[d];
  }
}

LLG_API int llg_kv_write(const void* k_new, const void* v_new, void* k_pages, void* v_pages,
                         const int* page_table, int table_width, int ring_pages, const int* positions,
                         const int* seq_of_token, const int* slots, const int* cu_tokens,
                         const int* len_before, int n_tokens, int nkv, int hd, int dtype,
                         cudaStream_t stream) {
  LLG_REQUIRE(n_tokens >= 0 && nkv > 0 && hd > 0 && ring_pages > 0 && table_width >= ring_pages,
              "kv_write: bad sizes");
  if (n_tokens == 0) return 0;
  const int warps = 4;
  const unsigned grid = (unsigned)(((long long)n_tokens * nkv + warps - 1) / warps);
  if (dtype == LLG_F32)
    kv_write_kernel<float><<<grid, warps * 32, 0, stream>>>(
        (const float*)k_new, (const float*)v_new, (float*)k_pages, (float*)v_pages, page_table, table_width,
        ring_pages, positions, seq_of_token, slots, cu_tokens, len_before, n_tokens, nkv, hd);
  else if (dtype == LLG_BF16)
    kv_write_kernel<__nv_bfloat16><<<grid, warps * 32, 0, stream>>>(
        (const __nv_bfloat16*)k_new, (const __nv_bfloat16*)v_new, (__nv_bfloat16*)k_pages,
        (__nv_bfloat16*)v_pages, page_table, table_width, ring_pages, positions, seq_of_token, slots,
        cu_tokens, len_before, n_tokens, nkv, hd);
  else
    return llg_fail("kv_write: unknown dtype %d", dtype);
  return llg_check_launch("kv_write");
}

// ---- SiLU gating --------------------------------------------------------------------

// The gate and up projections are stored as one matrix: the gate rows of all features, zero rows up
// to a multiple P of 128, then the up rows in the same way (the layout the tensor-core product's
// gated epilogue wants).  A product's output row therefore holds, for feature i, g at i and u at P + i:
// out[n][i] = silu(g) * u, silu(g) = g / (1 + exp(-g))  (Daisi.Llogos.Cpu/Silu.cs:9-16).
// `act`: what the gate passes: 2 silu, 1 the tanh form of gelu (the kinds of llg_act in common.cuh), -1: what `form` says.
template <typename IT, typename OT>
__global__ void silu_mul_kernel(const IT* __restrict__ gu, int n_partials, long long partial_stride,
                                OT* __restrict__ out, long long total, int inter, int width, int act, GateForm form) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
       idx += (long long)gridDim.x * blockDim.x) {
    const long long n = idx / inter;
    const int i = (int)(idx - n * inter);
    const IT* p = gu + n * width + i;
    float g = 0.f, u = 0.f;
    for (int s = 0; s < n_partials; ++s) {
      g += to_f32(p[s * partial_stride]);
      u += to_f32(p[s * partial_stride + width / 2]);
    }
    out[idx] = from_f32<OT>(act < 0 ? gate_form_of(form, g, u) : (act == 2 ? g / (1.0f + expf(-g)) : llg_act(act, g)) * u);
  }
}

static int gate_mul(const void* gu, int in_dtype, int n_partials, long long partial_stride, void* out,
                    int out_dtype, int n_tokens, int inter, int act, const GateForm& form, cudaStream_t stream);
static const GateForm SILU_FORM = {1.0f, 0.0f, INFINITY, 0.0f};

LLG_API int llg_silu_mul(const void* gu, int in_dtype, int n_partials, long long partial_stride, void* out,
                         int out_dtype, int n_tokens, int inter, cudaStream_t stream) {
  return gate_mul(gu, in_dtype, n_partials, partial_stride, out, out_dtype, n_tokens, inter, 2, SILU_FORM, stream);
}

// out[n][i] = act(g) * u with the gate's activation given by its kind (llg_act in common.cuh).
LLG_API int llg_gate_mul(const void* gu, int in_dtype, int n_partials, long long partial_stride, void* out,
                         int out_dtype, int n_tokens, int inter, int act, cudaStream_t stream) {
  LLG_REQUIRE(act >= 0 && act < LLG_ACT_KINDS, "gate_mul: activation kind %d is not known", act);
  return gate_mul(gu, in_dtype, n_partials, partial_stride, out, out_dtype, n_tokens, inter, act, SILU_FORM, stream);
}

// out[n][i] by a form of gating (GateForm in kernel_args.h).
LLG_API int llg_gate_form_mul(const void* gu, int in_dtype, int n_partials, long long partial_stride, void* out, int out_dtype,
                              int n_tokens, int inter, const GateForm* form, cudaStream_t stream) {
  return gate_mul(gu, in_dtype, n_partials, partial_stride, out, out_dtype, n_tokens, inter, -1, *form, stream);
}

static int gate_mul(const void* gu, int in_dtype, int n_partials, long long partial_stride, void* out,
                    int out_dtype, int n_tokens, int inter, int act, const GateForm& form, cudaStream_t stream) {
  LLG_REQUIRE(n_tokens >= 0 && inter > 0 && n_partials >= 1, "silu_mul: bad sizes");
  const long long total = (long long)n_tokens * inter;
  if (total == 0) return 0;
  const int width = ((inter + 127) / 128) * 256;
  const int threads = 256;
  long long blocks = (total + threads - 1) / threads;
  if (blocks > (long long)llg_sm_count() * 16) blocks = (long long)llg_sm_count() * 16;
#define LAUNCH(IT, OT)                                                                                          \
  silu_mul_kernel<IT, OT><<<(unsigned)blocks, threads, 0, stream>>>((const IT*)gu, n_partials, partial_stride, \
                                                                     (OT*)out, total, inter, width, act, form)
  if (in_dtype == LLG_F32 && out_dtype == LLG_F32) LAUNCH(float, float);
  else if (in_dtype == LLG_F32 && out_dtype == LLG_BF16) LAUNCH(float, __nv_bfloat16);
  else if (in_dtype == LLG_BF16 && out_dtype == LLG_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else return llg_fail("silu_mul: unsupported dtypes in=%d out=%d", in_dtype, out_dtype);
#undef LAUNCH
  return llg_check_launch("silu_mul");
}

// ---- small index updates ------------------------------------------------------------

// (No early launch of dependents here: kernels further down the step read the page table before
// they wait for their predecessor, so this kernel must be complete before any of them starts.)
__global__ void scatter_i32_kernel(int* __restrict__ dst, const int* __restrict__ idx,
                                   const int* __restrict__ val, int n) {
  pdl_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) dst[idx[i]] = val[i];
}

// dst[idx[i]] = val[i]: new page-table entries of a step, applied in one launch.
LLG_API int llg_scatter_i32(int* dst, const int* idx, const int* val, int n, cudaStream_t stream) {
  if (n <= 0) return 0;
  scatter_i32_kernel<<<(n + 255) / 256, 256, 0, stream>>>(dst, idx, val, n);
  return llg_check_launch("scatter_i32");
}

__global__ void gather_i32_kernel(int* __restrict__ dst, const int* __restrict__ src, const int* __restrict__ idx, int n) {
  pdl_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) dst[i] = src[idx[i]];
}

// dst[i] = src[idx[i]]: the tokens that a sampler left on the device become the next step's input.
LLG_API int llg_gather_i32(int* dst, const int* src, const int* idx, int n, cudaStream_t stream) {
  if (n <= 0) return 0;
  gather_i32_kernel<<<(n + 255) / 256, 256, 0, stream>>>(dst, src, idx, n);
  return llg_check_launch("gather_i32");
}

__global__ void zero_rows_kernel(unsigned char* __restrict__ base, const int* __restrict__ rows,
                                 long long row_bytes) {
  pdl_wait();
  unsigned char* p = base + (long long)rows[blockIdx.x] * row_bytes;
  for (long long i = threadIdx.x; i < row_bytes; i += blockDim.x) p[i] = 0;
}

// Zeroes the fixed-size state of the given slots (a sequence's state starts from zero).
LLG_API int llg_zero_rows(void* base, const int* rows, int n_rows, long long row_bytes, cudaStream_t stream) {
  if (n_rows <= 0 || row_bytes <= 0) return 0;
  zero_rows_kernel<<<n_rows, 256, 0, stream>>>((unsigned char*)base, rows, row_bytes);
  return llg_check_launch("zero_rows");
}

// ---- residual in several streams (hyper-connections) ----------------------------------

// See HyperNormArgs in kernel_args.h.  One block per output row; the read-out u stays in shared memory between the
// pass that updates the streams and the pass that writes the normalised row.
constexpr int HC_MAX = 16;    // most streams (the vector kernel holds up to HC_VEC_MAX of them in registers)
constexpr int HC_VEC_MAX = 8;

template <typename OT, typename WT>
__global__ void hc_add_rmsnorm_kernel(HyperNormArgs a) {
  pdl_launch_dependents();
  extern __shared__ float u_row[];               // [hidden]
  __shared__ float red[32];
  __shared__ float c_mix[HC_MAX * HC_MAX], c_write[HC_MAX], c_read[HC_MAX];
  const int S = a.n_streams;
  // the connection's weights are no result of this step: fetched while the kernel ahead still runs
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) c_mix[i] = a.branch ? a.mix[i] : 0.f;
  if (threadIdx.x < S) {
    c_write[threadIdx.x] = a.branch ? a.write[threadIdx.x] : 0.f;
    c_read[threadIdx.x] = a.read ? a.read[threadIdx.x] : 1.f;
  }
  pdl_wait();
  __syncthreads();
  const int j = blockIdx.x;
  const int r = a.rows ? a.rows[j] : j;
  const int hidden = a.hidden;
  float* base = a.streams + (long long)r * hidden;
  float ss = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    float x[HC_MAX];
#pragma unroll
    for (int s = 0; s < HC_MAX; ++s) x[s] = s < S ? base[s * a.stream_stride + i] : 0.f;
    if (a.branch) {
      const float* b = a.branch + (long long)r * hidden + i;
      float y = 0.f;
      for (int p = 0; p < a.n_partials; ++p) y += b[p * a.partial_stride];
      float nx[HC_MAX];
#pragma unroll
      for (int t = 0; t < HC_MAX; ++t) {
        float v = 0.f;
        if (t < S) {
#pragma unroll
          for (int s = 0; s < HC_MAX; ++s)
            if (s < S) v = fmaf(c_mix[s * S + t], x[s], v);
          v = fmaf(c_write[t], y, v);
          base[t * a.stream_stride + i] = v;
        }
        nx[t] = v;
      }
#pragma unroll
      for (int t = 0; t < HC_MAX; ++t) x[t] = nx[t];
    }
    float u = 0.f;
#pragma unroll
    for (int s = 0; s < HC_MAX; ++s)
      if (s < S) u = fmaf(c_read[s], x[s], u);
    u_row[i] = u;
    ss += u * u;
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)hidden + a.eps);
  OT* o = (OT*)a.out + (long long)j * hidden;
  const WT* w = (const WT*)a.weight;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) o[i] = from_f32<OT>(u_row[i] * inv * to_f32(w[i]));
}

// The same for rows whose length is a multiple of 4 and 16-byte aligned operands: 16-byte accesses, the read-out stays in
// registers between the two passes (VPT float4 per thread), and the partial sums of an element are asked for together.
// SMAX: the most streams an instance holds (its register arrays have that size).
template <typename OT, typename WT, int VPT, int SMAX>
__global__ void __launch_bounds__(512) hc_add_rmsnorm_vec4_kernel(HyperNormArgs a) {
  pdl_launch_dependents();
  __shared__ float red[32];
  __shared__ float c_mix[HC_MAX * HC_MAX], c_write[HC_MAX], c_read[HC_MAX];
  const int S = a.n_streams;
  const int nv = a.hidden >> 2;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) c_mix[i] = a.branch ? a.mix[i] : 0.f;
  if (threadIdx.x < S) {
    c_write[threadIdx.x] = a.branch ? a.write[threadIdx.x] : 0.f;
    c_read[threadIdx.x] = a.read ? a.read[threadIdx.x] : 1.f;
  }
  float wv[VPT][4];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < nv) vec_load4((const WT*)a.weight + 4 * i, wv[k]);
  }
  pdl_wait();
  __syncthreads();
  const int j = blockIdx.x;
  const int r = a.rows ? a.rows[j] : j;
  float4* base = reinterpret_cast<float4*>(a.streams + (long long)r * a.hidden);
  const long long ss4 = a.stream_stride >> 2, ps4 = a.partial_stride >> 2;
  float4 keep[VPT];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < nv) {
      float4 x[SMAX];
#pragma unroll
      for (int s = 0; s < SMAX; ++s) x[s] = s < S ? base[s * ss4 + i] : make_float4(0.f, 0.f, 0.f, 0.f);
      if (a.branch) {
        const float4* b = reinterpret_cast<const float4*>(a.branch + (long long)r * a.hidden) + i;
        float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
        int p = 0;
        for (; p + 4 <= a.n_partials; p += 4) {
          const float4 b0 = b[(p + 0) * ps4], b1 = b[(p + 1) * ps4], b2 = b[(p + 2) * ps4], b3 = b[(p + 3) * ps4];
          y.x += b0.x; y.y += b0.y; y.z += b0.z; y.w += b0.w;
          y.x += b1.x; y.y += b1.y; y.z += b1.z; y.w += b1.w;
          y.x += b2.x; y.y += b2.y; y.z += b2.z; y.w += b2.w;
          y.x += b3.x; y.y += b3.y; y.z += b3.z; y.w += b3.w;
        }
        for (; p < a.n_partials; ++p) {
          const float4 b0 = b[p * ps4];
          y.x += b0.x; y.y += b0.y; y.z += b0.z; y.w += b0.w;
        }
        float4 nx[SMAX];
#pragma unroll
        for (int t = 0; t < SMAX; ++t) {
          float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
          if (t < S) {
#pragma unroll
            for (int s = 0; s < SMAX; ++s) {
              if (s < S) {
                const float m = c_mix[s * S + t];
                v.x = fmaf(m, x[s].x, v.x); v.y = fmaf(m, x[s].y, v.y); v.z = fmaf(m, x[s].z, v.z); v.w = fmaf(m, x[s].w, v.w);
              }
            }
            const float wr = c_write[t];
            v.x = fmaf(wr, y.x, v.x); v.y = fmaf(wr, y.y, v.y); v.z = fmaf(wr, y.z, v.z); v.w = fmaf(wr, y.w, v.w);
            base[t * ss4 + i] = v;
          }
          nx[t] = v;
        }
#pragma unroll
        for (int t = 0; t < SMAX; ++t) x[t] = nx[t];
      }
#pragma unroll
      for (int s = 0; s < SMAX; ++s) {
        if (s < S) {
          const float rd = c_read[s];
          u.x = fmaf(rd, x[s].x, u.x); u.y = fmaf(rd, x[s].y, u.y); u.z = fmaf(rd, x[s].z, u.z); u.w = fmaf(rd, x[s].w, u.w);
        }
      }
    }
    keep[k] = u;
    ss += u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)a.hidden + a.eps);
  OT* o = (OT*)a.out + (long long)j * a.hidden;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < nv) {
      const float4 u = keep[k];
      const float y[4] = {u.x * inv * wv[k][0], u.y * inv * wv[k][1], u.z * inv * wv[k][2], u.w * inv * wv[k][3]};
      vec_store4(o + 4 * i, y);
    }
  }
}

LLG_API int llg_hc_max_streams() { return HC_MAX; }

LLG_API int llg_hc_add_rmsnorm(const HyperNormArgs* args, cudaStream_t stream) {
  const HyperNormArgs& a = *args;
  LLG_REQUIRE(a.n_out >= 0 && a.hidden > 0, "hc_add_rmsnorm: bad sizes n_out=%d hidden=%d", a.n_out, a.hidden);
  LLG_REQUIRE(a.n_streams >= 1 && a.n_streams <= HC_MAX, "hc_add_rmsnorm: %d streams, this kernel takes 1 to %d", a.n_streams, HC_MAX);
  LLG_REQUIRE(a.eps > 0.f, "hc_add_rmsnorm: eps must be positive");
  LLG_REQUIRE(!a.branch || (a.n_partials >= 1 && a.mix && a.write), "hc_add_rmsnorm: a branch needs partials, mix and write weights");
  if (a.n_out == 0) return 0;
  const size_t smem = (size_t)a.hidden * sizeof(float);
  LLG_REQUIRE(smem <= 200 * 1024, "hc_add_rmsnorm: rows of %d elements do not fit shared memory", a.hidden);
  int threads = a.hidden >= 2048 ? 512 : (a.hidden >= 512 ? 256 : 128);
  // vector path (as in llg_add_rmsnorm): few rows want many threads per row, many rows want the row in registers
  auto aligned = [](const void* p) { return ((uintptr_t)p & 15u) == 0; };
  const bool vec = a.hidden % 4 == 0 && a.stream_stride % 4 == 0 && a.partial_stride % 4 == 0 && aligned(a.streams) &&
                   aligned(a.branch) && aligned(a.weight) && aligned(a.out);
  int vpt = 1;
  if (vec) {
    const int nv = a.hidden / 4;
    // (at most 512 threads: a thread holds S float4 of the streams beside its part of the read-out)
    threads = a.n_out <= 256 ? (nv >= 512 ? 512 : (nv >= 256 ? 256 : 128)) : (nv >= 1024 ? 512 : 256);
    vpt = (nv + threads - 1) / threads;
    if (vpt > 4) {
      threads = 512;
      vpt = (nv + threads - 1) / threads;
    }
  }
  const bool vec_ok = vec && vpt <= 4 && a.n_streams <= HC_VEC_MAX;
#define LAUNCH_V(OT, WT, SM)                                                                                        \
  do {                                                                                                              \
    if (vpt <= 1) llg_launch(hc_add_rmsnorm_vec4_kernel<OT, WT, 1, SM>, a.n_out, threads, 0, stream, a);            \
    else if (vpt <= 2) llg_launch(hc_add_rmsnorm_vec4_kernel<OT, WT, 2, SM>, a.n_out, threads, 0, stream, a);       \
    else llg_launch(hc_add_rmsnorm_vec4_kernel<OT, WT, 4, SM>, a.n_out, threads, 0, stream, a);                     \
  } while (0)
#define LAUNCH(OT, WT)                                                                                              \
  do {                                                                                                              \
    if (vec_ok) {                                                                                                   \
      if (a.n_streams <= 2) LAUNCH_V(OT, WT, 2);                                                                    \
      else if (a.n_streams <= 4) LAUNCH_V(OT, WT, 4);                                                               \
      else LAUNCH_V(OT, WT, HC_VEC_MAX);                                                                            \
      break;                                                                                                        \
    }                                                                                                               \
    if (smem > 48 * 1024) {                                                                                         \
      cudaError_t e = cudaFuncSetAttribute(hc_add_rmsnorm_kernel<OT, WT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (e != cudaSuccess) return llg_fail("hc_add_rmsnorm: shared memory %zu: %s", smem, cudaGetErrorString(e));   \
    }                                                                                                               \
    llg_launch(hc_add_rmsnorm_kernel<OT, WT>, a.n_out, threads, smem, stream, a);                                   \
  } while (0)
  if (a.out_dtype == LLG_F32 && a.weight_dtype == LLG_F32) LAUNCH(float, float);
  else if (a.out_dtype == LLG_F32 && a.weight_dtype == LLG_BF16) LAUNCH(float, __nv_bfloat16);
  else if (a.out_dtype == LLG_BF16 && a.weight_dtype == LLG_F32) LAUNCH(__nv_bfloat16, float);
  else if (a.out_dtype == LLG_BF16 && a.weight_dtype == LLG_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else return llg_fail("hc_add_rmsnorm: unknown dtypes out=%d weight=%d", a.out_dtype, a.weight_dtype);
#undef LAUNCH
#undef LAUNCH_V
  return llg_check_launch("hc_add_rmsnorm");
}

// ---- queries, keys, values and gates from one product's row, norms over whole rows -------

// See QkvRowPrepArgs in kernel_args.h.  One block per token; the summed row stays in shared memory.
template <typename OT, typename WT>
__global__ void qkv_row_prep_kernel(QkvRowPrepArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float row[];                 // [q | k | v | gates]
  __shared__ float red[32];
  const int n = blockIdx.x;
  const int Q = a.nh * a.hd, K = a.nkv * a.hd, V = a.nkv * a.vd, G = a.gate_out ? a.nh : 0;
  const int W = Q + K + V + G;
  const float* src = a.qkvg + (long long)n * W;
  const WT* bias = (const WT*)a.bias;
  float ss_q = 0.f, ss_k = 0.f;
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    float v = 0.f;
    for (int p = 0; p < a.n_partials; ++p) v += src[p * a.partial_stride + i];
    if (bias && i < Q + K + V) v += to_f32(bias[i]);
    row[i] = v;
    if (i < Q) ss_q += v * v;
    else if (i < Q + K) ss_k += v * v;
  }
  ss_q = block_sum(ss_q, red);
  ss_k = block_sum(ss_k, red);
  __syncthreads();
  const float inv_q = a.q_norm_w ? 1.0f / sqrtf(ss_q / (float)Q + a.norm_eps) : 1.f;
  const float inv_k = (a.k_norm_w && K > 0) ? 1.0f / sqrtf(ss_k / (float)K + a.norm_eps) : 1.f;
  const WT* qw = (const WT*)a.q_norm_w;
  const WT* kw = (const WT*)a.k_norm_w;
  const int pos = a.positions[n];
  const bool to_pages = a.k_pages != nullptr;
  const int slot = to_pages ? a.slots[a.seq_of_token[n]] : 0;
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    const float v = row[i];
    if (i < Q) {
      ((OT*)a.q_out)[(long long)n * Q + i] = from_f32<OT>(qw ? v * inv_q * to_f32(qw[i]) : v);
    } else if (i < Q + K) {
      const int c = i - Q;
      const OT o = from_f32<OT>(kw ? v * inv_k * to_f32(kw[c]) : v);
      if (a.k_new) ((OT*)a.k_new)[(long long)n * K + c] = o;
      if (to_pages) {
        const long long r = kv_row(a.page_table, a.table_width, a.ring_pages, slot, pos, c / a.hd, a.nkv);
        ((OT*)a.k_pages)[r * a.hd + c % a.hd] = o;
      }
    } else if (i < Q + K + V) {
      const int c = i - Q - K;
      const OT o = from_f32<OT>(v);
      if (a.v_new) ((OT*)a.v_new)[(long long)n * V + c] = o;
      if (to_pages) {
        const long long r = kv_row(a.page_table, a.table_width, a.ring_pages, slot, pos, c / a.vd, a.nkv);
        ((OT*)a.v_pages)[r * a.vd + c % a.vd] = o;
      }
    } else {
      a.gate_out[(long long)n * a.nh + (i - Q - K - V)] = 1.0f / (1.0f + expf(-v));
    }
  }
}

// The same with 16-byte accesses, for head sizes and head counts that are multiples of 4 (every part of the row then
// starts and ends on a group of four) and 16-byte aligned operands.
__device__ __forceinline__ void vec_store4_any(float* p, const float (&v)[4]) { vec_store4(p, v); }
__device__ __forceinline__ void vec_store4_any(__nv_bfloat16* p, const float (&v)[4]) { vec_store4(p, v); }

template <typename OT, typename WT>
__global__ void qkv_row_prep_vec4_kernel(QkvRowPrepArgs a) {
  pdl_launch_dependents();
  extern __shared__ float row[];
  __shared__ float red[32];
  const int n = blockIdx.x;
  const int Q = a.nh * a.hd, K = a.nkv * a.hd, V = a.nkv * a.vd, G = a.gate_out ? a.nh : 0;
  const int W = Q + K + V + G, W4 = W >> 2;
  const WT* bias = (const WT*)a.bias;
  // positions, slots and the page table were written before this step's first kernel started
  const int pos = a.positions[n];
  const bool to_pages = a.k_pages != nullptr;
  const int slot = to_pages ? a.slots[a.seq_of_token[n]] : 0;
  pdl_wait();
  const float4* src = reinterpret_cast<const float4*>(a.qkvg + (long long)n * W);
  const long long ps4 = a.partial_stride >> 2;
  float ss_q = 0.f, ss_k = 0.f;
  for (int i4 = threadIdx.x; i4 < W4; i4 += blockDim.x) {
    const int i = i4 << 2;
    float4 v = src[i4];
    for (int p = 1; p < a.n_partials; ++p) {
      const float4 t = src[p * ps4 + i4];
      v.x += t.x; v.y += t.y; v.z += t.z; v.w += t.w;
    }
    if (bias && i < Q + K + V) {
      float b[4];
      vec_load4(bias + i, b);
      v.x += b[0]; v.y += b[1]; v.z += b[2]; v.w += b[3];
    }
    reinterpret_cast<float4*>(row)[i4] = v;
    const float sq = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    if (i < Q) ss_q += sq;
    else if (i < Q + K) ss_k += sq;
  }
  ss_q = block_sum(ss_q, red);
  ss_k = block_sum(ss_k, red);
  __syncthreads();
  const float inv_q = a.q_norm_w ? 1.0f / sqrtf(ss_q / (float)Q + a.norm_eps) : 1.f;
  const float inv_k = (a.k_norm_w && K > 0) ? 1.0f / sqrtf(ss_k / (float)K + a.norm_eps) : 1.f;
  const WT* qw = (const WT*)a.q_norm_w;
  const WT* kw = (const WT*)a.k_norm_w;
  for (int i4 = threadIdx.x; i4 < W4; i4 += blockDim.x) {
    const int i = i4 << 2;
    const float4 t = reinterpret_cast<const float4*>(row)[i4];
    float v[4] = {t.x, t.y, t.z, t.w};
    if (i < Q) {
      if (qw) {
        float w[4];
        vec_load4(qw + i, w);
#pragma unroll
        for (int c = 0; c < 4; ++c) v[c] = v[c] * inv_q * w[c];
      }
      vec_store4_any((OT*)a.q_out + (long long)n * Q + i, v);
    } else if (i < Q + K) {
      const int c0 = i - Q;
      if (kw) {
        float w[4];
        vec_load4(kw + c0, w);
#pragma unroll
        for (int c = 0; c < 4; ++c) v[c] = v[c] * inv_k * w[c];
      }
      if (a.k_new) vec_store4_any((OT*)a.k_new + (long long)n * K + c0, v);
      if (to_pages) {
        const long long r = kv_row(a.page_table, a.table_width, a.ring_pages, slot, pos, c0 / a.hd, a.nkv);
        vec_store4_any((OT*)a.k_pages + r * a.hd + c0 % a.hd, v);
      }
    } else if (i < Q + K + V) {
      const int c0 = i - Q - K;
      if (a.v_new) vec_store4_any((OT*)a.v_new + (long long)n * V + c0, v);
      if (to_pages) {
        const long long r = kv_row(a.page_table, a.table_width, a.ring_pages, slot, pos, c0 / a.vd, a.nkv);
        vec_store4_any((OT*)a.v_pages + r * a.vd + c0 % a.vd, v);
      }
    } else {
#pragma unroll
      for (int c = 0; c < 4; ++c) v[c] = 1.0f / (1.0f + expf(-v[c]));
      vec_store4(a.gate_out + (long long)n * a.nh + (i - Q - K - V), v);
    }
  }
}

LLG_API int llg_qkv_row_prep(const QkvRowPrepArgs* args, int out_dtype, cudaStream_t stream) {
  const QkvRowPrepArgs& a = *args;
  LLG_REQUIRE(a.n_tokens >= 0 && a.nh > 0 && a.nkv >= 0 && a.hd > 0 && a.vd > 0, "qkv_row_prep: bad sizes");
  LLG_REQUIRE(a.n_partials >= 1, "qkv_row_prep: n_partials must be >= 1");
  LLG_REQUIRE(!a.k_pages || (a.v_pages && a.page_table && a.slots && a.seq_of_token && a.ring_pages > 0),
              "qkv_row_prep: a cache write needs both page stores, page_table, slots and seq_of_token");
  LLG_REQUIRE((a.k_new == nullptr) == (a.v_new == nullptr), "qkv_row_prep: packed keys and values go together");
  if (a.n_tokens == 0) return 0;
  const long long w = (long long)a.nh * a.hd + (long long)a.nkv * (a.hd + a.vd) + (a.gate_out ? a.nh : 0);
  const size_t smem = (size_t)w * sizeof(float);
  LLG_REQUIRE(smem <= 200 * 1024, "qkv_row_prep: rows of %lld elements do not fit shared memory", w);
  auto aligned = [](const void* p) { return ((uintptr_t)p & 15u) == 0; };
  const bool vec = a.hd % 4 == 0 && a.vd % 4 == 0 && a.nh % 4 == 0 && a.partial_stride % 4 == 0 && aligned(a.qkvg) &&
                   aligned(a.bias) && aligned(a.q_norm_w) && aligned(a.k_norm_w) && aligned(a.q_out) && aligned(a.k_new) &&
                   aligned(a.v_new) && aligned(a.k_pages) && aligned(a.v_pages) && aligned(a.gate_out);
  // few tokens: the row's loads are the step's critical path, so more threads share them
  const int threads = vec ? (w >= 4096 && a.n_tokens <= 64 ? 1024 : (w >= 2048 && a.n_tokens <= 256) ? 512 : 256) : (w >= 2048 ? 512 : 256);
#define LAUNCH(OT, WT)                                                                                             \
  do {                                                                                                             \
    if (smem > 48 * 1024) {                                                                                        \
      cudaError_t e = cudaFuncSetAttribute(qkv_row_prep_kernel<OT, WT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (e == cudaSuccess) e = cudaFuncSetAttribute(qkv_row_prep_vec4_kernel<OT, WT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (e != cudaSuccess) return llg_fail("qkv_row_prep: shared memory %zu: %s", smem, cudaGetErrorString(e));    \
    }                                                                                                              \
    if (vec) llg_launch(qkv_row_prep_vec4_kernel<OT, WT>, a.n_tokens, threads, smem, stream, a);                   \
    else llg_launch(qkv_row_prep_kernel<OT, WT>, a.n_tokens, threads, smem, stream, a);                            \
  } while (0)
  if (out_dtype == LLG_F32 && a.w_dtype == LLG_F32) LAUNCH(float, float);
  else if (out_dtype == LLG_F32 && a.w_dtype == LLG_BF16) LAUNCH(float, __nv_bfloat16);
  else if (out_dtype == LLG_BF16 && a.w_dtype == LLG_F32) LAUNCH(__nv_bfloat16, float);
  else if (out_dtype == LLG_BF16 && a.w_dtype == LLG_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else return llg_fail("qkv_row_prep: unknown dtypes out=%d weights=%d", out_dtype, a.w_dtype);
#undef LAUNCH
  return llg_check_launch("qkv_row_prep");
}

// ---- activations of an ungated feed-forward ---------------------------------------------

// out[n][i] = act(sum of the partials of in[n][i]); the kinds are those of llg_act (common.cuh).

template <typename IT, typename OT>
__global__ void act_rows_kernel(const IT* __restrict__ in, int n_partials, long long partial_stride, OT* __restrict__ out,
                                long long total, int kind) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x) {
    float z = 0.f;
    for (int s = 0; s < n_partials; ++s) z += to_f32(in[s * partial_stride + idx]);
    out[idx] = from_f32<OT>(llg_act(kind, z));
  }
}

LLG_API int llg_act_rows(const void* in, int in_dtype, int n_partials, long long partial_stride, void* out, int out_dtype,
                         long long total, int kind, cudaStream_t stream) {
  LLG_REQUIRE(total >= 0 && n_partials >= 1 && kind >= 0 && kind <= 3, "act_rows: bad arguments");
  if (total == 0) return 0;
  const int threads = 256;
  long long blocks = (total + threads - 1) / threads;
  if (blocks > (long long)llg_sm_count() * 16) blocks = (long long)llg_sm_count() * 16;
#define LAUNCH(IT, OT) \
  llg_launch(act_rows_kernel<IT, OT>, (unsigned)blocks, threads, 0, stream, (const IT*)in, n_partials, partial_stride, (OT*)out, total, kind)
  if (in_dtype == LLG_F32 && out_dtype == LLG_F32) LAUNCH(float, float);
  else if (in_dtype == LLG_F32 && out_dtype == LLG_BF16) LAUNCH(float, __nv_bfloat16);
  else if (in_dtype == LLG_BF16 && out_dtype == LLG_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else return llg_fail("act_rows: unsupported dtypes in=%d out=%d", in_dtype, out_dtype);
#undef LAUNCH
  return llg_check_launch("act_rows");
}

// ---- a cap on logits ----------------------------------------------------------------------
// x <- cap * tanh(x / cap), in place (float32).
__global__ void tanh_cap_kernel(float* __restrict__ x, long long total, float cap) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x)
    x[i] = cap * tanhf(x[i] / cap);
}

LLG_API int llg_tanh_cap(float* x, long long total, float cap, cudaStream_t stream) {
  LLG_REQUIRE(total >= 0 && cap > 0.f, "tanh_cap: bad arguments (cap %g)", cap);
  if (total == 0) return 0;
  long long blocks = (total + 255) / 256;
  if (blocks > (long long)llg_sm_count() * 16) blocks = (long long)llg_sm_count() * 16;
  llg_launch(tanh_cap_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, x, total, cap);
  return llg_check_launch("tanh_cap");
}
