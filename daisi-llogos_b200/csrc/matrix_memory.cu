// A matrix memory per head with exponential gates and a running maximum (mLSTM), over the sequences of a step; the
// recurrence and the argument block are described in kernel_args.h (MatrixMemoryArgs).
//
//   matrix_memory        : a block owns (sequence or piece, head, a run of `cols` columns of the head's state S).  S lies
//                          in registers: thread (sl, j) keeps rows sl * R .. sl * R + R - 1 of column j.  Tokens are taken
//                          MEM_BATCH at a time: their q, k, v and gate arguments are summed from the product's partials
//                          into shared memory, the batch's running maxima come from a scan over its lanes (max and plus),
//                          and the walk through the batch needs no barrier.  n, one vector per head, is kept by every
//                          block of the head (its product with q is needed by all columns).  Read-outs, denominators and,
//                          where a block has all columns of the head, the norm and the output gate are done together for
//                          the batch, a warp per token.
//   matrix_memory_join   : walks a sequence's pieces and leaves in each piece's carry the state it starts from.
//   matrix_memory_finish : norm and output gate of heads that were cut into several runs of columns.
//
// All of it is float32 arithmetic, whatever the output type.
#include "common.cuh"
#include "kernel_args.h"

LLG_API const char* llg_last_error() { return g_llg_error; }

namespace {

constexpr int MEM_BATCH = 16;
constexpr int JOIN_BATCH = 8;

__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float y) { return fminf(y, 0.f) - log1pf(expf(-fabsf(y))); }

__device__ __forceinline__ long long carry_stride(const MatrixMemoryArgs& a) {
  return (long long)a.dim * a.vdim + a.dim + LLG_MEMORY_CARRY_EXTRA;
}

// the tokens of a block's piece: [lo, hi)
__device__ __forceinline__ void piece_range(const MatrixMemoryArgs& a, int b, int piece, bool pieces, int& lo, int& hi, int& t_end) {
  const int t_begin = a.cu_tokens[b];
  t_end = a.cu_tokens[b + 1];
  lo = t_begin;
  hi = t_end;
  if (pieces) {
    lo = t_begin + piece * a.piece;
    if (lo > t_end) lo = t_end;
    hi = (piece == a.pieces - 1 || lo + a.piece > t_end) ? t_end : lo + a.piece;
  }
}

// MODE 0: a sequence from its state to its state; 1: a piece from zero, only its state is wanted; 2: a piece from the
// state the join left.
template <typename OT, int MODE, int R, int TH>
__global__ void __launch_bounds__(TH, 512 / TH) matrix_memory_kernel(MatrixMemoryArgs a, int runs) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float smem[];
  __shared__ float s_i[MEM_BATCH], s_f[MEM_BATCH];
  const int h = blockIdx.x, piece = blockIdx.y / runs, run = blockIdx.y % runs, b = blockIdx.z;
  const int dim = a.dim, vdim = a.vdim, cols = a.cols;
  const int slices = TH / cols;
  const int dp = slices * R;                  // padded length of a q, k or n row
  const int sl = threadIdx.x / cols, j = threadIdx.x - sl * cols;
  const int c0 = run * cols;                  // first column of this block
  const int nc = min(cols, vdim - c0);        // its columns
  const bool active = sl < slices && j < nc;
  const bool whole = runs == 1;
  float* sq = smem;                           // [MEM_BATCH][dp]
  float* sk = sq + MEM_BATCH * dp;            // [MEM_BATCH][dp]
  float* pn = sk + MEM_BATCH * dp;            // [MEM_BATCH][dp]: n * q, element by element
  float* sn = pn + MEM_BATCH * dp;            // [dp]: n
  float* sv = sn + dp;                        // [MEM_BATCH][cols]
  float* po = sv + MEM_BATCH * cols;          // [MEM_BATCH][slices][cols]
  int lo, hi, t_end;
  piece_range(a, b, piece, MODE != 0, lo, hi, t_end);
  if (MODE == 2 && lo >= hi) return;
  const int slot = a.slots[b];
  float* gs = a.state_s + ((long long)slot * a.nh + h) * dim * vdim;
  float* gn = a.state_n + ((long long)slot * a.nh + h) * dim;
  float* gm = a.state_m + (long long)slot * a.nh + h;
  float* cr = MODE != 0 ? a.carry + (((long long)b * a.pieces + piece) * a.nh + h) * carry_stride(a) : nullptr;
  const float* src_s = MODE == 0 ? gs : cr;
  const float* src_n = MODE == 0 ? gn : cr + (long long)dim * vdim;
  float S[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = sl * R + r;
    S[r] = (MODE != 1 && active && i < dim) ? src_s[(long long)i * vdim + c0 + j] : 0.f;
  }
  for (int i = threadIdx.x; i < dp; i += TH) sn[i] = (MODE != 1 && i < dim) ? src_n[i] : 0.f;
  float m = MODE == 1 ? -INFINITY : MODE == 0 ? *gm : cr[(long long)dim * vdim + dim + 2];
  float f_total = 0.f;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  OT* out = (OT*)a.out;
  for (int n0 = lo; n0 < hi; n0 += MEM_BATCH) {
    const int nb = min(MEM_BATCH, hi - n0);
    const float* rows = a.rows + (long long)n0 * a.row_width;
    auto summed = [&](int t, int col) {
      const float* p = rows + (long long)t * a.row_width + col;
      float v = p[0];
      for (int s = 1; s < a.n_partials; ++s) v += p[s * a.partial_stride];
      return v;
    };
    for (int idx = threadIdx.x; idx < nb * dp; idx += TH) {
      const int t = idx / dp, i = idx - t * dp;
      sk[idx] = i < dim ? summed(t, a.k_col + h * dim + i) : 0.f;
      if (MODE != 1) sq[idx] = i < dim ? summed(t, a.q_col + h * dim + i) * a.q_scale : 0.f;
    }
    for (int idx = threadIdx.x; idx < nb * cols; idx += TH) {
      const int t = idx / cols, c = idx - t * cols;
      sv[idx] = c < nc ? summed(t, a.v_col + h * vdim + c0 + c) : 0.f;
    }
    if (threadIdx.x < 2 * nb) {
      const int t = threadIdx.x >> 1;
      if (threadIdx.x & 1) s_f[t] = log_sigmoid(capped(summed(t, a.f_col + h) + (a.f_bias ? a.f_bias[h] : 0.f), a.gate_cap));
      else s_i[t] = capped(summed(t, a.i_col + h) + (a.i_bias ? a.i_bias[h] : 0.f), a.gate_cap);
    }
    __syncthreads();
    // every warp works out the batch's maxima: lane t's pair (f, i) stands for m -> max(m + f, i), and pairs compose
    float keep = 0.f, take = 0.f, low = 0.f, m_last;
    {
      const float f = lane < nb ? s_f[lane] : 0.f, i = lane < nb ? s_i[lane] : -INFINITY;
      float fa = f, ib = i;
#pragma unroll
      for (int o = 1; o < MEM_BATCH; o <<= 1) {
        const float pf = __shfl_up_sync(0xffffffffu, fa, o), pi = __shfl_up_sync(0xffffffffu, ib, o);
        if (lane >= o) {
          ib = fmaxf(pi + fa, ib);
          fa += pf;
        }
      }
      const float mt = fmaxf(fa + m, ib);
      float before = __shfl_up_sync(0xffffffffu, mt, 1);
      if (lane == 0) before = m;
      keep = expf(f + before - mt);
      take = expf(i - mt);
      low = expf(-mt);
      m_last = __shfl_sync(0xffffffffu, mt, nb - 1);
      f_total += __shfl_sync(0xffffffffu, fa, nb - 1);
    }
    for (int t = 0; t < nb; ++t) {
      const float kp = __shfl_sync(0xffffffffu, keep, t), tk = __shfl_sync(0xffffffffu, take, t);
      if (active) {
        const float vj = sv[t * cols + j] * tk;
        const float4* kt = reinterpret_cast<const float4*>(sk + t * dp + sl * R);
        const float4* qt = reinterpret_cast<const float4*>(sq + t * dp + sl * R);
        float o = 0.f;
#pragma unroll
        for (int r4 = 0; r4 < R / 4; ++r4) {
          const float4 kk = kt[r4];
          S[4 * r4] = fmaf(kp, S[4 * r4], kk.x * vj);
          S[4 * r4 + 1] = fmaf(kp, S[4 * r4 + 1], kk.y * vj);
          S[4 * r4 + 2] = fmaf(kp, S[4 * r4 + 2], kk.z * vj);
          S[4 * r4 + 3] = fmaf(kp, S[4 * r4 + 3], kk.w * vj);
          if (MODE != 1) {
            const float4 qq = qt[r4];
            o = fmaf(S[4 * r4], qq.x, o);
            o = fmaf(S[4 * r4 + 1], qq.y, o);
            o = fmaf(S[4 * r4 + 2], qq.z, o);
            o = fmaf(S[4 * r4 + 3], qq.w, o);
          }
        }
        if (MODE != 1) po[(t * slices + sl) * cols + j] = o;
      }
      for (int i = threadIdx.x; i < dp; i += TH) {       // a row of n has one owner
        const float v = fmaf(kp, sn[i], tk * sk[t * dp + i]);
        sn[i] = v;
        if (MODE != 1) pn[t * dp + i] = v * sq[t * dp + i];
      }
    }
    m = m_last;
    if (MODE != 1) {
      __syncthreads();
      for (int t = warp; t < nb; t += TH / 32) {
        float dot = 0.f;
        for (int i = lane; i < dp; i += 32) dot += pn[t * dp + i];
        dot = warp_sum(dot);
        const float inv_den = 1.0f / (fmaxf(fabsf(dot), __shfl_sync(0xffffffffu, low, t)) + a.denom_eps);
        float ss = 0.f;
        const long long at = ((long long)(n0 + t) * a.nh + h) * vdim + c0;
        for (int c = lane; c < nc; c += 32) {
          float o = po[t * slices * cols + c];
          for (int s = 1; s < slices; ++s) o += po[(t * slices + s) * cols + c];
          o *= inv_den;
          if (whole) po[t * slices * cols + c] = o;
          else a.raw[at + c] = o;
          ss = fmaf(o, o, ss);
        }
        if (!whole) continue;
        ss = warp_sum(ss);
        const float inv = 1.0f / sqrtf(ss / (float)vdim + a.eps);
        for (int c = lane; c < vdim; c += 32) {
          const float g = summed(t, a.g_col + h * vdim + c);
          out[at + c] = from_f32<OT>(po[t * slices * cols + c] * inv * a.norm_w[h * vdim + c] / (1.0f + expf(-g)));
        }
      }
    }
    __syncthreads();
  }
  // the state it ends with
  const bool last = MODE == 2 && hi == t_end;
  if (MODE != 2 || last) {
    float* dst = MODE == 1 ? cr : gs;
    if (active) {
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const int i = sl * R + r;
        if (i < dim) dst[(long long)i * vdim + c0 + j] = S[r];
      }
    }
    if (run == 0) {
      // other blocks of this head may still have to read n and m of the state: cut heads put theirs aside
      const bool aside = MODE == 0 && !whole;
      float* nx = aside ? a.next + ((long long)b * a.nh + h) * (dim + 1) : nullptr;
      float* dn = MODE == 1 ? cr + (long long)dim * vdim : aside ? nx : gn;
      for (int i = threadIdx.x; i < dim; i += TH) dn[i] = sn[i];
      if (threadIdx.x == 0) {
        if (MODE == 1) {
          cr[(long long)dim * vdim + dim] = f_total;
          cr[(long long)dim * vdim + dim + 1] = m;
        } else if (aside) {
          nx[dim] = m;
        } else {
          *gm = m;
        }
      }
    }
  }
}

// One thread per element of (S, n): walks the pieces, S -> e^{F + m - m'} S + e^{m_p - m'} S_p with m' = max(F + m, m_p), where
// F and m_p are the piece's sum of log forget gates and its own maximum.  A piece's entry is replaced by what it starts from.
__global__ void __launch_bounds__(256) matrix_memory_join_kernel(MatrixMemoryArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, b = blockIdx.z;
  const int ns = a.dim * a.vdim, total = ns + a.dim;
  const int e = blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= total) return;
  const int slot = a.slots[b];
  float S = e < ns ? a.state_s[((long long)slot * a.nh + h) * ns + e] : a.state_n[((long long)slot * a.nh + h) * a.dim + e - ns];
  float m = a.state_m[(long long)slot * a.nh + h];
  const long long step = (long long)a.nh * carry_stride(a);
  float* cr = a.carry + ((long long)b * a.pieces * a.nh + h) * carry_stride(a);
  for (int p0 = 0; p0 < a.pieces; p0 += JOIN_BATCH, cr += JOIN_BATCH * step) {
    float reached[JOIN_BATCH], F[JOIN_BATCH], mp[JOIN_BATCH];
#pragma unroll
    for (int k = 0; k < JOIN_BATCH; ++k) {
      if (p0 + k < a.pieces) {
        reached[k] = cr[k * step + e];
        F[k] = cr[k * step + total];
        mp[k] = cr[k * step + total + 1];
      }
    }
#pragma unroll
    for (int k = 0; k < JOIN_BATCH; ++k) {
      if (p0 + k < a.pieces) {
        cr[k * step + e] = S;
        if (e == 0) cr[k * step + total + 2] = m;
        const float mn = fmaxf(F[k] + m, mp[k]);
        S = expf(F[k] + m - mn) * S + expf(mp[k] - mn) * reached[k];
        m = mn;
      }
    }
  }
}

// Heads that were cut into runs of columns: a warp per (token, head) norms and gates raw; the blocks behind those put n and m
// of the sequences into the state (where `next` is given).
template <typename OT>
__global__ void __launch_bounds__(128) matrix_memory_finish_kernel(MatrixMemoryArgs a, int head_blocks) {
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if ((int)blockIdx.x >= head_blocks) {
    const int item = (blockIdx.x - head_blocks) * 4 + warp;
    if (item >= a.n_seqs * a.nh) return;
    const int b = item / a.nh, h = item % a.nh, slot = a.slots[b];
    const float* nx = a.next + (long long)item * (a.dim + 1);
    for (int i = lane; i < a.dim; i += 32) a.state_n[((long long)slot * a.nh + h) * a.dim + i] = nx[i];
    if (lane == 0) a.state_m[(long long)slot * a.nh + h] = nx[a.dim];
    return;
  }
  const long long item = (long long)blockIdx.x * 4 + warp;
  if (item >= (long long)a.n_tokens * a.nh) return;
  const long long n = item / a.nh;
  const int h = (int)(item % a.nh), vdim = a.vdim;
  const float* o = a.raw + item * vdim;
  float ss = 0.f;
  for (int c = lane; c < vdim; c += 32) ss = fmaf(o[c], o[c], ss);
  ss = warp_sum(ss);
  const float inv = 1.0f / sqrtf(ss / (float)vdim + a.eps);
  const float* gr = a.rows + n * a.row_width + a.g_col + h * vdim;
  OT* out = (OT*)a.out + item * vdim;
  for (int c = lane; c < vdim; c += 32) {
    float g = gr[c];
    for (int s = 1; s < a.n_partials; ++s) g += gr[s * a.partial_stride + c];
    out[c] = from_f32<OT>(o[c] * inv * a.norm_w[h * vdim + c] / (1.0f + expf(-g)));
  }
}

// Rows of a column per thread (4, 8, 16 or 32; 0: more than that) and shared memory of a block of `threads` threads.
size_t memory_smem(int dim, int cols, int threads, int* r_out) {
  const int slices = threads / cols;
  if (slices == 0) {
    *r_out = 0;
    return 0;
  }
  const int rows = (dim + slices - 1) / slices;
  const int r = threads == 512 ? 32 : rows <= 4 ? 4 : rows <= 8 ? 8 : rows <= 16 ? 16 : 32;      // (512 threads have one form)
  *r_out = rows <= 32 ? r : 0;
  const size_t dp = (size_t)slices * r;
  return (3 * MEM_BATCH * dp + dp + (size_t)MEM_BATCH * cols + (size_t)MEM_BATCH * slices * cols) * sizeof(float);
}

// The threads of a block that can own `cols` columns of `dim` rows: 256, else 512, else 0.
int memory_threads(int dim, int cols) {
  for (int th = 256; th <= 512; th *= 2) {
    int r = 0;
    const size_t smem = memory_smem(dim, cols, th, &r);
    if (r > 0 && smem <= 220 * 1024) return th;
  }
  return 0;
}

template <typename K>
int memory_attr(K kernel, size_t smem) {
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return llg_fail("matrix_memory: shared memory %zu: %s", smem, cudaGetErrorString(e));
  }
  return 0;
}

template <typename OT, int R, int TH>
int memory_run(const MatrixMemoryArgs& a, size_t smem, cudaStream_t stream) {
  const int runs = (a.vdim + a.cols - 1) / a.cols;
  if (!a.carry) {
    if (memory_attr(matrix_memory_kernel<OT, 0, R, TH>, smem)) return 1;
    llg_launch(matrix_memory_kernel<OT, 0, R, TH>, dim3(a.nh, runs, a.n_seqs), dim3(TH), smem, stream, a, runs);
  } else {
    if (memory_attr(matrix_memory_kernel<OT, 1, R, TH>, smem) || memory_attr(matrix_memory_kernel<OT, 2, R, TH>, smem)) return 1;
    const dim3 grid(a.nh, (unsigned)(a.pieces * runs), a.n_seqs);
    llg_launch(matrix_memory_kernel<OT, 1, R, TH>, grid, dim3(TH), smem, stream, a, runs);
    llg_launch(matrix_memory_join_kernel, dim3((a.dim * a.vdim + a.dim + 255) / 256, a.nh, a.n_seqs), dim3(256), 0, stream, a);
    llg_launch(matrix_memory_kernel<OT, 2, R, TH>, grid, dim3(TH), smem, stream, a, runs);
  }
  if (runs > 1) {
    const long long head_blocks = ((long long)a.n_tokens * a.nh + 3) / 4;
    const long long blocks = head_blocks + (a.carry ? 0 : (a.n_seqs * a.nh + 3) / 4);
    LLG_REQUIRE(blocks < 2147483647LL, "matrix_memory: too many tokens");
    llg_launch(matrix_memory_finish_kernel<OT>, dim3((unsigned)blocks), dim3(128), 0, stream, a, (int)head_blocks);
  }
  return llg_check_launch("matrix_memory");
}

template <typename OT>
int memory_launch(const MatrixMemoryArgs& a, cudaStream_t stream) {
  int r = 0;
  const int th = memory_threads(a.dim, a.cols);
  const size_t smem = memory_smem(a.dim, a.cols, th, &r);
  if (th == 256) {
    if (r == 4) return memory_run<OT, 4, 256>(a, smem, stream);
    if (r == 8) return memory_run<OT, 8, 256>(a, smem, stream);
    if (r == 16) return memory_run<OT, 16, 256>(a, smem, stream);
    return memory_run<OT, 32, 256>(a, smem, stream);
  }
  return memory_run<OT, 32, 512>(a, smem, stream);
}

}  // namespace

// 1 when a block can own `cols` columns of a head with a state of `dim` rows.
LLG_API int llg_matrix_memory_fits(int dim, int cols) {
  return dim > 0 && cols > 0 && memory_threads(dim, cols) > 0;
}

LLG_API int llg_matrix_memory(const MatrixMemoryArgs* args, int max_count, cudaStream_t stream) {
  const MatrixMemoryArgs& a = *args;
  LLG_REQUIRE(a.n_seqs >= 0 && a.n_tokens >= 0 && a.nh > 0 && a.dim > 0 && a.vdim > 0 && a.n_partials >= 1, "matrix_memory: bad sizes");
  LLG_REQUIRE(a.n_seqs <= 65535 && a.nh <= 65535, "matrix_memory: too many sequences or heads");
  LLG_REQUIRE(a.gate_cap > 0.f && a.eps > 0.f, "matrix_memory: gate cap %g, eps %g", a.gate_cap, a.eps);
  LLG_REQUIRE(a.cols > 0 && a.cols <= a.vdim && llg_matrix_memory_fits(a.dim, a.cols),
              "matrix_memory: %d columns of a state of %d rows do not fit a block", a.cols, a.dim);
  const int ends[6] = {a.q_col + a.nh * a.dim, a.k_col + a.nh * a.dim, a.v_col + a.nh * a.vdim, a.g_col + a.nh * a.vdim,
                       a.i_col + a.nh, a.f_col + a.nh};
  const int starts[6] = {a.q_col, a.k_col, a.v_col, a.g_col, a.i_col, a.f_col};
  for (int i = 0; i < 6; ++i)
    LLG_REQUIRE(starts[i] >= 0 && ends[i] <= a.row_width, "matrix_memory: columns %d to %d of rows of %d", starts[i], ends[i], a.row_width);
  const int runs = (a.vdim + a.cols - 1) / a.cols;
  LLG_REQUIRE(runs == 1 || (a.raw && (a.carry || a.next)), "matrix_memory: a head in several runs of columns needs raw and next");
  if (a.carry)
    LLG_REQUIRE(a.pieces >= 1 && a.piece >= 1 && (long long)a.pieces * runs <= 65535 && (long long)a.pieces * a.piece >= max_count,
                "matrix_memory: %d pieces of %d tokens do not hold a sequence of %d", a.pieces, a.piece, max_count);
  if (a.n_seqs == 0 || a.n_tokens == 0) return 0;
  if (a.out_dtype == LLG_F32) return memory_launch<float>(a, stream);
  if (a.out_dtype == LLG_BF16) return memory_launch<__nv_bfloat16>(a, stream);
  return llg_fail("matrix_memory: unknown output type %d", a.out_dtype);
}
