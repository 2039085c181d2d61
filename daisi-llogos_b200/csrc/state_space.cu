// State-space recurrences with a scalar decay per head and step (argument block in kernel_args.h: StateSpaceArgs), and the
// RMS norm in equal parts that stands behind them.
//
//   state_space_walk : any sizes, float32 arithmetic.  A block owns some columns of one head's state in registers and walks a
//                      sequence's tokens in order, sixteen at a time: their B, C, x and step sizes are fetched together,
//                      the walk through a batch needs no barrier, and the batch's read-outs are added up together.  A
//                      decode step is a batch of one token; the state is then what bounds the kernel, and it is requested
//                      before the kernel ahead has finished (no kernel near it writes it).
//   state_space_mma  : prompt steps in bfloat16.  A block owns some columns of one head's state as the accumulators of tensor-core
//                      products and walks a sequence in chunks of 64 tokens.  With a_t the running sum of the chunk's
//                      log decays and S0 the state before the chunk,
//                        y_t = e^{a_t} C_t S0 + sum_{s <= t} e^{a_t - a_s} d_s (C_t . B_s) x_s
//                        S   = e^{a_end} S0 + sum_s B_s (e^{a_end - a_s} d_s x_s)^T
//                      B, C and x are bfloat16 as the convolution left them and enter the products exactly; what is float32
//                      (the state, and the factors made of decays and step sizes) enters as a sum of two bfloat16 numbers,
//                      each with a product of its own, so a factor keeps 16 bits and the sums are float32.
//   part_rmsnorm     : rows in equal parts, each divided by its own root mean square, times a weight.
#include "common.cuh"
#include "kernel_args.h"

LLG_API const char* llg_last_error() { return g_llg_error; }

namespace {

typedef __nv_bfloat16 bf16;

constexpr int SS_THREADS = 256;
constexpr int SS_BATCH = 16;             // tokens fetched together by the walk
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float softplus_f(float v) { return v > 20.f ? v : log1pf(expf(v)); }

// The step size of head h at packed token n.
__device__ __forceinline__ float step_size(const StateSpaceArgs& a, int h, int n) {
  const float* p = a.rows + (long long)n * a.row_width + a.dt_col + h;
  float v = p[0];
  for (int s = 1; s < a.n_partials; ++s) v += p[s * a.partial_stride];
  return softplus_f(v + a.dt_bias[h]);
}

// Shared memory: B [SS_BATCH][np] | C [SS_BATCH][np] | x [SS_BATCH][cols] | partial read-outs [SS_BATCH][slices][cols], np = slices * R.
template <typename XT, int R>
__global__ void __launch_bounds__(SS_THREADS) state_space_walk_kernel(StateSpaceArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float smem[];
  __shared__ float s_step[SS_BATCH], s_decay[SS_BATCH];
  const int runs = (a.vdim + a.cols - 1) / a.cols;
  const int h = blockIdx.x / runs, c0 = (blockIdx.x - h * runs) * a.cols, b = blockIdx.y;
  const int nc = min(a.cols, a.vdim - c0);
  const int slices = SS_THREADS / a.cols, np = slices * R;
  const int sl = threadIdx.x / a.cols, j = threadIdx.x - sl * a.cols;
  const bool active = sl < slices && j < nc;
  float* sb = smem;
  float* sc = sb + SS_BATCH * np;
  float* sx = sc + SS_BATCH * np;
  float* po = sx + SS_BATCH * a.cols;
  float* gstate = a.state + ((long long)a.slots[b] * a.nh + h) * a.n_state * a.vdim + c0;
  float2 S[R / 2];
#pragma unroll
  for (int r = 0; r < R / 2; ++r) {
    const int i = sl * R + 2 * r;
    S[r].x = active && i < a.n_state ? gstate[(long long)i * a.vdim + j] : 0.f;
    S[r].y = active && i + 1 < a.n_state ? gstate[(long long)(i + 1) * a.vdim + j] : 0.f;
  }
  const float rate = -expf(a.a_log[h]), skip = a.d_skip[h];
  const int lo = a.cu_tokens[b], hi = a.cu_tokens[b + 1];
  const int mixed_w = a.nh * a.vdim + 2 * a.groups * a.n_state;
  const int b_col = a.nh * a.vdim + h / (a.nh / a.groups) * a.n_state, c_col = b_col + a.groups * a.n_state;
  pdl_wait();
  for (int n0 = lo; n0 < hi; n0 += SS_BATCH) {
    const int nb = min(SS_BATCH, hi - n0);
    if (threadIdx.x < nb) {
      const float d = step_size(a, h, n0 + threadIdx.x);
      s_step[threadIdx.x] = d;
      s_decay[threadIdx.x] = expf(rate * d);
    }
    const XT* rows = (const XT*)a.mixed + (long long)n0 * mixed_w;
    for (int idx = threadIdx.x; idx < nb * np; idx += SS_THREADS) {
      const int t = idx / np, i = idx - t * np;
      const XT* row = rows + (long long)t * mixed_w;
      sb[idx] = i < a.n_state ? to_f32(row[b_col + i]) : 0.f;
      sc[idx] = i < a.n_state ? to_f32(row[c_col + i]) : 0.f;
    }
    for (int idx = threadIdx.x; idx < nb * nc; idx += SS_THREADS) {
      const int t = idx / nc, c = idx - t * nc;
      sx[t * a.cols + c] = to_f32(rows[(long long)t * mixed_w + h * a.vdim + c0 + c]);
    }
    __syncthreads();
    if (active) {
      for (int t = 0; t < nb; ++t) {
        const float e = s_decay[t], xj = s_step[t] * sx[t * a.cols + j];
        const float2 e2 = make_float2(e, e), x2 = make_float2(xj, xj);
        const float4* bt = reinterpret_cast<const float4*>(sb + t * np + sl * R);
        const float4* ct = reinterpret_cast<const float4*>(sc + t * np + sl * R);
        float2 o2[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
#pragma unroll
        for (int r4 = 0; r4 < R / 4; ++r4) {
          const float4 bb = bt[r4], cc = ct[r4];
          S[2 * r4] = __ffma2_rn(make_float2(bb.x, bb.y), x2, __fmul2_rn(e2, S[2 * r4]));
          S[2 * r4 + 1] = __ffma2_rn(make_float2(bb.z, bb.w), x2, __fmul2_rn(e2, S[2 * r4 + 1]));
          o2[0] = __ffma2_rn(S[2 * r4], make_float2(cc.x, cc.y), o2[0]);
          o2[1] = __ffma2_rn(S[2 * r4 + 1], make_float2(cc.z, cc.w), o2[1]);
        }
        po[(t * slices + sl) * a.cols + j] = (o2[0].x + o2[0].y) + (o2[1].x + o2[1].y);
      }
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < nb * nc; idx += SS_THREADS) {
      const int t = idx / nc, c = idx - t * nc;
      float o = skip * sx[t * a.cols + c];
      for (int s = 0; s < slices; ++s) o += po[(t * slices + s) * a.cols + c];
      const int col = h * a.vdim + c0 + c;
      if (a.z_col >= 0) {
        const float* zp = a.rows + (long long)(n0 + t) * a.row_width + a.z_col + col;
        float z = zp[0];
        for (int s = 1; s < a.n_partials; ++s) z += zp[s * a.partial_stride];
        o *= z / (1.0f + expf(-z));
      }
      a.out[(long long)(n0 + t) * a.nh * a.vdim + col] = o;
    }
    __syncthreads();
  }
  if (active && lo < hi) {
#pragma unroll
    for (int r = 0; r < R / 2; ++r) {
      const int i = sl * R + 2 * r;
      if (i < a.n_state) gstate[(long long)i * a.vdim + j] = S[r].x;
      if (i + 1 < a.n_state) gstate[(long long)(i + 1) * a.vdim + j] = S[r].y;
    }
  }
}

// ---- the chunked form on the tensor cores --------------------------------------------------------------------------

constexpr int CH = 64;                   // tokens of a chunk
constexpr int MM_THREADS = 256;
constexpr float LEAST_LOG2 = -160.f;     // a decay below 2^-160 forgets everything; bounding it keeps the running sums short

__device__ __forceinline__ uint32_t smem_at(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

__device__ __forceinline__ void copy16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;                             // 0: the 16 bytes are filled with zeros, src is not read
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}

__device__ __forceinline__ void ldm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldm4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float exp2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two float32 numbers as two pairs of bfloat16 whose sum they are to 16 bits
__device__ __forceinline__ void split2(float v0, float v1, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(v0, v1);
  const __nv_bfloat162 l = __floats2bfloat162_rn(v0 - __low2float(h), v1 - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

// Two groups of four warps share a chunk; warp w of either group owns tokens 16 w .. of it.
//   inside : C B^T, the factors, their product with x, and the output (with what the other group hands over, D x and the gate)
//   across : C S0 for the chunk's tokens, handed over in shared memory as the registers hold it, then the state's update;
//            warp w owns every fourth 16 rows of the state
// One barrier of the block a chunk; the groups meet once more where the read-out is handed over.  The next chunk's rows are
// requested at a chunk's start, its step sizes and their running sums are worked out beside the chunk.
//
// MT: 16-row tiles of the state per warp (n_state <= 64 MT); NV: 8-column tiles (8 NV columns of vdim a block).
// Shared memory (bfloat16): two stages of B [CH][n_state + 8], C the same, x [CH][8 NV + 8]; the state as two parts
// [2][n_state][8 NV + 8], or the read-out of S0 in float32 [4][NV][32][4]; the weighed x as two parts [2][CH][8 NV + 8].
// bfloat16 places of the state's parts, in whose place the read-out is handed over once they have been read
__host__ __device__ constexpr int state_halves(int n_state, int cols) {
  return 2 * n_state * (cols + 8) > 2 * CH * cols ? 2 * n_state * (cols + 8) : 2 * CH * cols;
}

__device__ __forceinline__ void group_sync(int id) { asm volatile("bar.sync %0, 128;" ::"r"(id) : "memory"); }

template <int MT, int NV>
__global__ void __launch_bounds__(MM_THREADS, MT <= 2 && NV <= 4 ? 2 : 1) state_space_mma_kernel(StateSpaceArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) unsigned char raw_smem[];
  // per token of a chunk: the step size d, the running sum of log2 decays a, d 2^{a_end - a} (what its x weighs in the state behind
  // the chunk), and d 2^{E - a} with E the sum at the end of its sixteen tokens (its part of a factor for later tokens)
  __shared__ float s_step[2][CH], s_log[2][CH], s_last[2][CH], s_part[2][CH];
  constexpr int VS = 8 * NV, LDV = VS + 8;
  const int N = a.n_state, LDN = N + 8, NT = N / 16;
  bf16* stage0 = reinterpret_cast<bf16*>(raw_smem);
  const int stage_halves = 2 * CH * LDN + CH * LDV;
  bf16* state_sm = stage0 + 2 * stage_halves;
  bf16* wx = state_sm + state_halves(N, VS);
  float4* handed = reinterpret_cast<float4*>(state_sm);
  const int tid = threadIdx.x, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const bool across = tid >= 128;
  const int warp = (tid >> 5) & 3;                       // inside its group
  const int runs = a.vdim / VS;
  const int h = blockIdx.x / runs, c0 = (blockIdx.x - h * runs) * VS, b = blockIdx.y;
  const int lo = a.cu_tokens[b], hi = a.cu_tokens[b + 1];
  if (lo >= hi) return;
  const int mixed_w = a.nh * a.vdim + 2 * a.groups * N, inner = a.nh * a.vdim;
  const int b_col = inner + h / (a.nh / a.groups) * N, c_col = b_col + a.groups * N, x_col = h * a.vdim + c0;
  float* gstate = a.state + ((long long)a.slots[b] * a.nh + h) * N * a.vdim + c0;
  float S[MT][NV][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int row = (warp + 4 * mt) * 16 + g;
      const bool in = across && warp + 4 * mt < NT;
      const float* p = gstate + (long long)row * a.vdim + v * 8 + 2 * t4;
      const float2 u = in ? *reinterpret_cast<const float2*>(p) : make_float2(0.f, 0.f);
      const float2 w = in ? *reinterpret_cast<const float2*>(p + 8LL * a.vdim) : make_float2(0.f, 0.f);
      S[mt][v][0] = u.x; S[mt][v][1] = u.y; S[mt][v][2] = w.x; S[mt][v][3] = w.y;
    }
  const float rate2 = -expf(a.a_log[h]) * LOG2E, skip = a.d_skip[h], dt_bias = a.dt_bias[h];
  pdl_wait();

  const bf16* mixed = (const bf16*)a.mixed;
  const int per = N / 8;                                 // 16-byte pieces of a row of B or C
  const int t_first = tid / per, c_first = tid - t_first * per, t_step = MM_THREADS / per, c_step = MM_THREADS - t_step * per;
  auto load_chunk = [&](int n0, int stage) {
    bf16* base = stage0 + stage * stage_halves;
    if (n0 + CH <= hi && c_step == 0) {
      // a whole chunk whose pieces divide among the threads: the same piece of every t_step-th row
      const bf16* src = mixed + (long long)(n0 + t_first) * mixed_w + c_first * 8;
      const long long src_step = (long long)t_step * mixed_w;
      uint32_t dst = smem_at(base + t_first * LDN + c_first * 8);
      const uint32_t dst_step = (uint32_t)(t_step * LDN * 2), to_c = (uint32_t)(CH * LDN * 2);
      for (int t = t_first; t < CH; t += t_step) {
        copy16(dst, src + b_col, true);
        copy16(dst + to_c, src + c_col, true);
        src += src_step;
        dst += dst_step;
      }
    } else {
      for (int t = t_first, c = c_first; t < CH;) {
        const bool valid = n0 + t < hi;
        const bf16* row = mixed + (long long)(valid ? n0 + t : lo) * mixed_w + c * 8;
        copy16(smem_at(base + t * LDN + c * 8), row + b_col, valid);
        copy16(smem_at(base + (CH + t) * LDN + c * 8), row + c_col, valid);
        t += t_step;
        c += c_step;
        if (c >= per) { c -= per; ++t; }
      }
    }
#pragma unroll
    for (int idx = tid; idx < CH * NV; idx += MM_THREADS) {
      const int t = idx / NV, c = idx - t * NV;
      const bool valid = n0 + t < hi;
      copy16(smem_at(base + 2 * CH * LDN + t * LDV + c * 8), mixed + (long long)(valid ? n0 + t : lo) * mixed_w + x_col + c * 8, valid);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // the first warp: the step sizes' arguments of tokens n0 + 2 lane and n0 + 2 lane + 1, and what becomes of them
  float arg0 = 0.f, arg1 = 0.f;
  auto fetch_steps = [&](int n0) {
    const int n = n0 + 2 * lane;
    const float* p = a.rows + a.dt_col + h;
    // nothing is added to the first loads' results here: they would be waited for
    arg0 = n < hi ? p[(long long)n * a.row_width] : 0.f;
    arg1 = n + 1 < hi ? p[(long long)(n + 1) * a.row_width] : 0.f;
    for (int s = 1; s < a.n_partials; ++s) {
      if (n < hi) arg0 += p[s * a.partial_stride + (long long)n * a.row_width];
      if (n + 1 < hi) arg1 += p[s * a.partial_stride + (long long)(n + 1) * a.row_width];
    }
  };
  auto put_steps = [&](int n0, int buf) {
    // tokens past the end: no step and no decay, so they change nothing
    const int n = n0 + 2 * lane;
    const float d0 = n < hi ? softplus_f(arg0 + dt_bias) : 0.f, d1 = n + 1 < hi ? softplus_f(arg1 + dt_bias) : 0.f;
    const float l0 = fmaxf(rate2 * d0, LEAST_LOG2), l1 = fmaxf(rate2 * d1, LEAST_LOG2);
    float incl = l0 + l1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += up;
    }
    const float up1 = __shfl_up_sync(0xffffffffu, incl, 1), log0 = (lane ? up1 : 0.f) + l0;
    const float end = __shfl_sync(0xffffffffu, incl, 31), block_end = __shfl_sync(0xffffffffu, incl, lane | 7);
    *reinterpret_cast<float2*>(&s_step[buf][2 * lane]) = make_float2(d0, d1);
    *reinterpret_cast<float2*>(&s_log[buf][2 * lane]) = make_float2(log0, incl);
    *reinterpret_cast<float2*>(&s_last[buf][2 * lane]) = make_float2(d0 * exp2_fast(end - log0), d1 * exp2_fast(end - incl));
    *reinterpret_cast<float2*>(&s_part[buf][2 * lane]) = make_float2(d0 * exp2_fast(block_end - log0), d1 * exp2_fast(block_end - incl));
  };
  load_chunk(lo, 0);
  if (tid < 32) {
    fetch_steps(lo);
    put_steps(lo, 0);
  }
  int stage = 0;
  for (int n0 = lo; n0 < hi; n0 += CH, stage ^= 1) {
    const bool more = n0 + CH < hi;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                       // the chunk and its sums of logs are there; the other stage may be written again
    if (more) load_chunk(n0 + CH, stage ^ 1);
    const bf16* Bs = stage0 + stage * stage_halves;
    const bf16* Cs = Bs + CH * LDN;
    const bf16* Xs = Cs + CH * LDN;
    const float *slog = s_log[stage], *sstep = s_step[stage];
    const int r0 = warp * 16 + g, r1 = r0 + 8;
    const float a0 = slog[r0], a1 = slog[r1];
    if (across) {
      // the state before the chunk, in two parts, for the group's products with C
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        if (warp + 4 * mt < NT) {
#pragma unroll
          for (int v = 0; v < NV; ++v) {
            bf16* p = state_sm + ((warp + 4 * mt) * 16 + g) * LDV + v * 8 + 2 * t4;
            uint32_t h0, l0, h1, l1;
            split2(S[mt][v][0], S[mt][v][1], h0, l0);
            split2(S[mt][v][2], S[mt][v][3], h1, l1);
            *reinterpret_cast<uint32_t*>(p) = h0;
            *reinterpret_cast<uint32_t*>(p + 8 * LDV) = h1;
            *reinterpret_cast<uint32_t*>(p + N * LDV) = l0;
            *reinterpret_cast<uint32_t*>(p + N * LDV + 8 * LDV) = l1;
          }
        }
      }
      group_sync(1);
      float y[NV][4];
#pragma unroll
      for (int v = 0; v < NV; ++v)
#pragma unroll
        for (int e = 0; e < 4; ++e) y[v][e] = 0.f;
#pragma unroll 4
      for (int kk = 0; kk < NT; ++kk) {
        uint32_t ca[4];
        ldm4(ca, smem_at(Cs + (warp * 16 + (lane & 15)) * LDN + kk * 16 + (lane >> 4) * 8));
#pragma unroll
        for (int v = 0; v < NV; ++v) {
          uint32_t sb[4];                  // both parts of 16 rows and 8 columns of the state
          ldm4_trans(sb, smem_at(state_sm + ((lane >> 4) * N + kk * 16 + (lane & 15)) * LDV + v * 8));
          mma16816(y[v], ca, sb[0], sb[1]);
          mma16816(y[v], ca, sb[2], sb[3]);
        }
      }
      const float e0 = exp2_fast(a0), e1 = exp2_fast(a1);
      group_sync(1);                       // nobody reads the state's parts any more: the read-out takes their place
#pragma unroll
      for (int v = 0; v < NV; ++v) handed[(warp * NV + v) * 32 + lane] = make_float4(y[v][0] * e0, y[v][1] * e0, y[v][2] * e1, y[v][3] * e1);
      asm volatile("bar.arrive 2, 256;" ::: "memory");
      // x times e^{a_end - a_s} d_s in two parts, then S = e^{a_end} S0 + B^T (weighed x)
      const float log_end = slog[CH - 1];
      for (int idx = tid - 128; idx < CH * NV * 4; idx += 128) {
        const int s = idx / (NV * 4), c = (idx - s * (NV * 4)) * 2;
        const float w = s_last[stage][s];
        const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(Xs + s * LDV + c);
        uint32_t hi2, lo2;
        split2(w * __low2float(x), w * __high2float(x), hi2, lo2);
        *reinterpret_cast<uint32_t*>(wx + s * LDV + c) = hi2;
        *reinterpret_cast<uint32_t*>(wx + (CH + s) * LDV + c) = lo2;
      }
      const float e_end = exp2_fast(log_end);
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int v = 0; v < NV; ++v)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[mt][v][e] *= e_end;
      group_sync(1);
#pragma unroll
      for (int kk = 0; kk < CH / 16; ++kk) {
        uint32_t ba[MT][4];                // B^T
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
          if (warp + 4 * mt < NT)
            ldm4_trans(ba[mt], smem_at(Bs + (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * LDN + (warp + 4 * mt) * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
        for (int v = 0; v < NV; ++v) {
          uint32_t wb[4];                  // both parts of the weighed x of 16 tokens
          ldm4_trans(wb, smem_at(wx + ((lane >> 4) * CH + kk * 16 + (lane & 15)) * LDV + v * 8));
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            if (warp + 4 * mt < NT) {
              mma16816(S[mt][v], ba[mt], wb[0], wb[1]);
              mma16816(S[mt][v], ba[mt], wb[2], wb[3]);
            }
          }
        }
      }
      continue;
    }
    // asked for now, used at the end: the gates' arguments and (first warp) the next chunk's step sizes
    float z[NV][4];
    if (a.z_col >= 0) {
      const float* zp = a.rows + (long long)(n0 + r0) * a.row_width + a.z_col + x_col + 2 * t4;
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        z[v][0] = n0 + r0 < hi ? zp[v * 8] : 0.f;
        z[v][1] = n0 + r0 < hi ? zp[v * 8 + 1] : 0.f;
        z[v][2] = n0 + r1 < hi ? zp[8LL * a.row_width + v * 8] : 0.f;
        z[v][3] = n0 + r1 < hi ? zp[8LL * a.row_width + v * 8 + 1] : 0.f;
      }
      for (int s = 1; s < a.n_partials; ++s) {
        zp += a.partial_stride;
#pragma unroll
        for (int v = 0; v < NV; ++v) {
          if (n0 + r0 < hi) { z[v][0] += zp[v * 8]; z[v][1] += zp[v * 8 + 1]; }
          if (n0 + r1 < hi) { z[v][2] += zp[8LL * a.row_width + v * 8]; z[v][3] += zp[8LL * a.row_width + v * 8 + 1]; }
        }
      }
    }
    if (more && warp == 0) fetch_steps(n0 + CH);
    // C B^T for this warp's tokens (columns up to its own last token)
    float G[8][4], y[NV][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) G[i][e] = 0.f;
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
      for (int e = 0; e < 4; ++e) y[v][e] = 0.f;
#pragma unroll 4
    for (int kk = 0; kk < NT; ++kk) {
      uint32_t ca[4];
      ldm4(ca, smem_at(Cs + (warp * 16 + (lane & 15)) * LDN + kk * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int sp = 0; sp < 4; ++sp) {
        if (sp <= warp) {
          uint32_t bb[4];
          ldm4(bb, smem_at(Bs + (sp * 16 + (lane & 7) + ((lane >> 4) << 3)) * LDN + kk * 16 + ((lane >> 3) & 1) * 8));
          mma16816(G[2 * sp], ca, bb[0], bb[1]);
          mma16816(G[2 * sp + 1], ca, bb[2], bb[3]);
        }
      }
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      if (kk > warp) continue;
      uint32_t ah[4], al[4];
      if (kk < warp) {
        // sixteen earlier tokens: 2^{a_t - a_s} d_s as 2^{a_t - E} times the token's part up to E, neither above d_s
        const float block_end = slog[kk * 16 + 15], e0 = exp2_fast(a0 - block_end), e1 = exp2_fast(a1 - block_end);
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const float2 q = *reinterpret_cast<const float2*>(&s_part[stage][kk * 16 + half * 8 + 2 * t4]);
          const float(&gv)[4] = G[2 * kk + half];
          split2(gv[0] * (e0 * q.x), gv[1] * (e0 * q.y), ah[2 * half], al[2 * half]);
          split2(gv[2] * (e1 * q.x), gv[3] * (e1 * q.y), ah[2 * half + 1], al[2 * half + 1]);
        }
      } else
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int s = kk * 16 + half * 8 + 2 * t4;
        const float2 la = *reinterpret_cast<const float2*>(slog + s), d = *reinterpret_cast<const float2*>(sstep + s);
        const float(&gv)[4] = G[2 * kk + half];
        const float m00 = s <= r0 ? gv[0] * (exp2_fast(a0 - la.x) * d.x) : 0.f;
        const float m01 = s + 1 <= r0 ? gv[1] * (exp2_fast(a0 - la.y) * d.y) : 0.f;
        const float m10 = s <= r1 ? gv[2] * (exp2_fast(a1 - la.x) * d.x) : 0.f;
        const float m11 = s + 1 <= r1 ? gv[3] * (exp2_fast(a1 - la.y) * d.y) : 0.f;
        split2(m00, m01, ah[2 * half], al[2 * half]);
        split2(m10, m11, ah[2 * half + 1], al[2 * half + 1]);
      }
#pragma unroll
      for (int v = 0; v < NV; v += 2) {    // x of 16 tokens and up to 16 columns
        uint32_t xb[4];
        ldm4_trans(xb, smem_at(Xs + (kk * 16 + (lane & 15)) * LDV + (v + (NV > 1 ? lane >> 4 : 0)) * 8));
        mma16816(y[v], ah, xb[0], xb[1]);
        mma16816(y[v], al, xb[0], xb[1]);
        if (NV > 1) {
          mma16816(y[(v + 1) % NV], ah, xb[2], xb[3]);
          mma16816(y[(v + 1) % NV], al, xb[2], xb[3]);
        }
      }
    }
    if (more && warp == 0) put_steps(n0 + CH, stage ^ 1);
    asm volatile("bar.sync 2, 256;" ::: "memory");       // what the state before the chunk gives is there
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const __nv_bfloat162 x0 = *reinterpret_cast<const __nv_bfloat162*>(Xs + r0 * LDV + v * 8 + 2 * t4);
      const __nv_bfloat162 x1 = *reinterpret_cast<const __nv_bfloat162*>(Xs + r1 * LDV + v * 8 + 2 * t4);
      const float4 q = handed[(warp * NV + v) * 32 + lane];
      float o[4] = {fmaf(skip, __low2float(x0), y[v][0] + q.x), fmaf(skip, __high2float(x0), y[v][1] + q.y),
                    fmaf(skip, __low2float(x1), y[v][2] + q.z), fmaf(skip, __high2float(x1), y[v][3] + q.w)};
      if (a.z_col >= 0) {
#pragma unroll
        for (int e = 0; e < 4; ++e) o[e] *= __fdividef(z[v][e], 1.0f + __expf(-z[v][e]));
      }
      float* dst = a.out + (long long)(n0 + r0) * inner + x_col + v * 8 + 2 * t4;
      if (n0 + r0 < hi) *reinterpret_cast<float2*>(dst) = make_float2(o[0], o[1]);
      if (n0 + r1 < hi) *reinterpret_cast<float2*>(dst + 8LL * inner) = make_float2(o[2], o[3]);
    }
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
    if (across && warp + 4 * mt < NT) {
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        float* p = gstate + (long long)((warp + 4 * mt) * 16 + g) * a.vdim + v * 8 + 2 * t4;
        *reinterpret_cast<float2*>(p) = make_float2(S[mt][v][0], S[mt][v][1]);
        *reinterpret_cast<float2*>(p + 8LL * a.vdim) = make_float2(S[mt][v][2], S[mt][v][3]);
      }
    }
  }
}

// ---- RMS norm in equal parts -------------------------------------------------------------------------------------------

// out[n][i] = x[n][i] / sqrt(mean over i's part of x[n]^2 + eps) * weight[i].  A block per (row, part); four elements an access and
// the part in registers where it is short enough and its length a multiple of four.
constexpr int PN_VPT = 4;

__device__ __forceinline__ void store_four(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store_four(bf16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 t;
  t.x = *reinterpret_cast<const uint32_t*>(&lo);
  t.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = t;
}

template <typename OT>
__global__ void part_rmsnorm_kernel(const float* __restrict__ x, const float* __restrict__ weight, OT* __restrict__ out, int parts,
                                    int per, float eps, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const long long row = blockIdx.x / parts;
  const int part = (int)(blockIdx.x - row * parts);
  const float* src = x + (row * parts + part) * per;
  const float* w = weight + (long long)part * per;
  OT* dst = out + (row * parts + part) * per;
  float ss = 0.f;
  if (vec) {
    float4 keep[PN_VPT];
#pragma unroll
    for (int k = 0; k < PN_VPT; ++k) {
      const int i = 4 * (threadIdx.x + k * blockDim.x);
      keep[k] = i < per ? *reinterpret_cast<const float4*>(src + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += keep[k].x * keep[k].x + keep[k].y * keep[k].y + keep[k].z * keep[k].z + keep[k].w * keep[k].w;
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)per + eps);
#pragma unroll
    for (int k = 0; k < PN_VPT; ++k) {
      const int i = 4 * (threadIdx.x + k * blockDim.x);
      if (i < per) {
        const float4 u = *reinterpret_cast<const float4*>(w + i);
        store_four(dst + i, make_float4(keep[k].x * inv * u.x, keep[k].y * inv * u.y, keep[k].z * inv * u.z, keep[k].w * inv * u.w));
      }
    }
    return;
  }
  for (int i = threadIdx.x; i < per; i += blockDim.x) ss = fmaf(src[i], src[i], ss);
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)per + eps);
  for (int i = threadIdx.x; i < per; i += blockDim.x) dst[i] = from_f32<OT>(src[i] * inv * w[i]);
}

template <typename K>
int allow_smem(K kernel, size_t smem) {
  if (smem > 40 * 1024) {                   // the kernels' static shared memory counts toward the 48 KB that need no asking
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return llg_fail("state_space: shared memory %zu: %s", smem, cudaGetErrorString(e));
  }
  return 0;
}

// Columns a block of the walk owns, rows a thread keeps of a column, and the shared memory (0 where a head does not fit).
struct WalkShape {
  int cols, rows;
  size_t smem;
};
WalkShape walk_shape(int n_state, int vdim) {
  for (int cols = vdim < SS_THREADS ? vdim : SS_THREADS; cols >= 1; cols = cols > 1 ? (cols + 1) / 2 : 0) {
    const int slices = SS_THREADS / cols, need = (n_state + slices - 1) / slices;
    if (need <= 32) {
      const int r = need <= 4 ? 4 : need <= 8 ? 8 : need <= 16 ? 16 : 32;
      const size_t smem = (size_t)SS_BATCH * (2 * slices * r + cols + slices * cols) * sizeof(float);
      return smem <= 200 * 1024 ? WalkShape{cols, r, smem} : WalkShape{0, 0, 0};
    }
  }
  return WalkShape{0, 0, 0};
}

size_t mma_smem(int n_state, int cols) {
  return (size_t)(2 * (2 * CH * (n_state + 8) + CH * (cols + 8)) + state_halves(n_state, cols) + 2 * CH * (cols + 8)) * sizeof(bf16);
}
// Columns a block owns: as many as fit (fewer columns repeat C B^T more often), fewer where that would leave too many
// multiprocessors without a block.  0: none fit.
int mma_cols(int n_state, int vdim, long long heads) {
  int last = 0;
  for (int cols = 64; cols >= 8; cols /= 2) {
    if (vdim % cols || mma_smem(n_state, cols) > 220 * 1024) continue;
    last = cols;
    if (heads * (vdim / cols) * 4 >= 3LL * llg_sm_count()) return cols;
  }
  return last;
}

int check_args(const StateSpaceArgs& a, const char* what) {
  LLG_REQUIRE(a.n_seqs >= 0 && a.n_tokens >= 0 && a.nh > 0 && a.groups > 0 && a.n_state > 0 && a.vdim > 0 && a.n_partials >= 1,
              "%s: bad sizes", what);
  LLG_REQUIRE(a.nh % a.groups == 0, "%s: %d heads do not split into %d groups", what, a.nh, a.groups);
  LLG_REQUIRE(a.n_seqs <= 65535, "%s: %d sequences in a step (at most 65535)", what, a.n_seqs);
  LLG_REQUIRE(a.dt_col >= 0 && a.dt_col + a.nh <= a.row_width && (a.z_col < 0 || a.z_col + a.nh * a.vdim <= a.row_width),
              "%s: columns outside a row of %d", what, a.row_width);
  return 0;
}

}  // namespace

// 1 when the walk takes a head's state of these sizes.
LLG_API int llg_state_space_fits(int n_state, int vdim) { return n_state > 0 && vdim > 0 && walk_shape(n_state, vdim).cols > 0; }

// 1 when the tensor-core form takes it (bfloat16, prompt steps).
LLG_API int llg_state_space_mma_fits(int n_state, int vdim) {
  return n_state > 0 && n_state % 16 == 0 && n_state <= 256 && mma_cols(n_state, vdim, 1) > 0;
}

LLG_API int llg_state_space_walk(const StateSpaceArgs* args, cudaStream_t stream) {
  StateSpaceArgs a = *args;
  if (check_args(a, "state_space_walk")) return 1;
  const WalkShape w = walk_shape(a.n_state, a.vdim);
  LLG_REQUIRE(w.cols > 0, "state_space_walk: a head's state of %d x %d does not fit a block", a.n_state, a.vdim);
  if (a.n_seqs == 0 || a.n_tokens == 0) return 0;
  a.cols = w.cols;
  const dim3 grid(a.nh * ((a.vdim + w.cols - 1) / w.cols), a.n_seqs);
#define WALK(XT, R)                                                              \
  do {                                                                           \
    if (allow_smem(state_space_walk_kernel<XT, R>, w.smem)) return 1;            \
    llg_launch(state_space_walk_kernel<XT, R>, grid, dim3(SS_THREADS), w.smem, stream, a); \
  } while (0)
#define WALK_R(XT)                   \
  do {                               \
    if (w.rows == 4) WALK(XT, 4);    \
    else if (w.rows == 8) WALK(XT, 8); \
    else if (w.rows == 16) WALK(XT, 16); \
    else WALK(XT, 32);               \
  } while (0)
  if (a.mixed_dtype == LLG_F32) WALK_R(float);
  else if (a.mixed_dtype == LLG_BF16) WALK_R(bf16);
  else return llg_fail("state_space_walk: unknown type %d", a.mixed_dtype);
#undef WALK_R
#undef WALK
  return llg_check_launch("state_space_walk");
}

LLG_API int llg_state_space_mma(const StateSpaceArgs* args, cudaStream_t stream) {
  StateSpaceArgs a = *args;
  if (check_args(a, "state_space_mma")) return 1;
  LLG_REQUIRE(a.mixed_dtype == LLG_BF16 && llg_state_space_mma_fits(a.n_state, a.vdim),
              "state_space_mma: a head's state of %d x %d (bfloat16, rows in steps of 16 up to 256, columns in steps of 8)", a.n_state, a.vdim);
  LLG_REQUIRE(((uintptr_t)a.mixed & 15u) == 0 && ((uintptr_t)a.state & 15u) == 0 && ((uintptr_t)a.out & 15u) == 0,
              "state_space_mma: operands must be 16-byte aligned");
  if (a.n_seqs == 0 || a.n_tokens == 0) return 0;
  if (a.cols == 0) a.cols = mma_cols(a.n_state, a.vdim, (long long)a.nh * a.n_seqs);
  LLG_REQUIRE((a.cols == 8 || a.cols == 16 || a.cols == 32 || a.cols == 64) && a.vdim % a.cols == 0 && mma_smem(a.n_state, a.cols) <= 220 * 1024,
              "state_space_mma: %d columns a block of a state of %d x %d", a.cols, a.n_state, a.vdim);
  const size_t smem = mma_smem(a.n_state, a.cols);
  const dim3 grid(a.nh * (a.vdim / a.cols), a.n_seqs);
#define GO(MT, NV)                                                                   \
  do {                                                                               \
    if (allow_smem(state_space_mma_kernel<MT, NV>, smem)) return 1;                  \
    llg_launch(state_space_mma_kernel<MT, NV>, grid, dim3(MM_THREADS), smem, stream, a); \
  } while (0)
#define GO_M(NV)                       \
  do {                                 \
    if (a.n_state <= 64) GO(1, NV);    \
    else if (a.n_state <= 128) GO(2, NV); \
    else GO(4, NV);                    \
  } while (0)
  if (a.cols == 64) GO_M(8);
  else if (a.cols == 32) GO_M(4);
  else if (a.cols == 16) GO_M(2);
  else GO_M(1);
#undef GO_M
#undef GO
  return llg_check_launch("state_space_mma");
}

LLG_API int llg_part_rmsnorm(const float* x, const float* weight, void* out, int out_dtype, int rows, int width, int parts, float eps,
                             cudaStream_t stream) {
  LLG_REQUIRE(rows >= 0 && width > 0 && parts > 0 && width % parts == 0 && eps > 0.f, "part_rmsnorm: %d elements in %d equal parts, eps %g",
              width, parts, eps);
  LLG_REQUIRE((long long)rows * parts < 2147483647LL, "part_rmsnorm: too many rows");
  if (rows == 0) return 0;
  const int per = width / parts;
  // few rows: a thread per four elements; many: as many as keep the part in registers
  int threads = (per + 3) / 4;
  if (rows > 64) threads = (threads + 1) / 2;
  threads = (threads + 31) / 32 * 32;
  threads = threads < 32 ? 32 : threads > 1024 ? 1024 : threads;
  const int vec = per % 4 == 0 && per <= 4 * PN_VPT * threads && ((uintptr_t)x % 16) == 0 && ((uintptr_t)weight % 16) == 0 && ((uintptr_t)out % 16) == 0;
  const dim3 grid((unsigned)(rows * (long long)parts));
  if (out_dtype == LLG_F32) llg_launch(part_rmsnorm_kernel<float>, grid, dim3(threads), 0, stream, x, weight, (float*)out, parts, per, eps, vec);
  else if (out_dtype == LLG_BF16) llg_launch(part_rmsnorm_kernel<bf16>, grid, dim3(threads), 0, stream, x, weight, (bf16*)out, parts, per, eps, vec);
  else return llg_fail("part_rmsnorm: unknown output type %d", out_dtype);
  return llg_check_launch("part_rmsnorm");
}
