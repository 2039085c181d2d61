// Attention whose scores are capped and mixed over the heads (see attention_mix.cu for the mathematics), on the tensor
// cores, for bfloat16 storage and head sizes that are multiples of 16 up to 128 (keys and values each).  Products of
// queries and keys and of weights and values are mma.sync m16n8k16 with float32 accumulation; scores, cap, mixture (plain
// float32 multiply-adds) and softmax are float32; weights are rounded to bfloat16 only as the operand of the second
// product.
//
//   attn_mix_prefill_mma : a cluster of C blocks takes BQ queries of all heads, every block H / C of the heads.  Per key tile a
//                          block computes its heads' scores and writes them into the shared memory of every block of the
//                          cluster; behind a cluster barrier each block mixes all heads' scores into its own heads' and
//                          goes on with their softmax and values by itself.
//   attn_mix_decode_mma  : one new token per sequence; a block takes a share of a sequence's keys for all heads (the
//                          partial results are joined by attn_decode_reduce).
//
// Shared-memory rows of bfloat16 are padded by 16 bytes (conflict-free ldmatrix), rows of scores by 8 floats.
#include "common.cuh"
#include "kernel_args.h"
#include "attention_reduce.cuh"

LLG_API const char* llg_last_error() { return g_llg_error; }

namespace {

typedef __nv_bfloat16 bf16;
constexpr int MT = 512;                 // threads of a block (16 warps)
constexpr int MW = MT / 32;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// 2^d for a whole number d <= 0 (or -inf), exactly
__device__ __forceinline__ float pow2_whole(float d) { return d < -126.f ? 0.f : __int_as_float((127 + (int)d) << 23); }

// cap tanh(s / cap) as cap (1 - 2 / (1 + e^(2 s / cap))): its absolute error is a rounding of cap, which is what counts ahead
// of an exponential.  An infinite exponential gives cap, one of zero -cap.
__device__ __forceinline__ float capped(float s, float cap, float two_over_cap) {
  return cap > 0.f ? cap - __fdividef(2.0f * cap, 1.0f + fminf(__expf(s * two_over_cap), 1e30f)) : s;
}

__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ uint32_t cluster_rank() {
  uint32_t r;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
  return r;
}
// the address of this block's shared-memory address `a` in block `rank` of the cluster
__device__ __forceinline__ uint32_t cluster_addr(uint32_t a, uint32_t rank) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(a), "r"(rank));
  return r;
}
__device__ __forceinline__ void cluster_store2(uint32_t a, float x, float y) {
  asm volatile("st.shared::cluster.v2.f32 [%0], {%1, %2};" ::"r"(a), "f"(x), "f"(y) : "memory");
}

// How a prompt step's work is cut: C blocks per cluster with hc heads each, qt sub-tiles of 16 queries, kt keys per tile.
struct MixCut {
  int c, hc, qt, kt, kvn;               // kvn: key/value heads that a block's heads can reach
  size_t smem;
};

__host__ __device__ inline int mix_score_stride(int kt) { return kt + 8; }

// ---- prompt steps --------------------------------------------------------------------------------

// Shared memory: Q [hc][BQ][rsk], K [kvn][KT][rsk], V [kvn][KT][rsv] (bytes per row rsk = 2 hd + 16, rsv = 2 vd + 16), scores
// [nh][BQ][KT + 8] floats, the mixture's columns T [nh][hc8] (hc8 = hc rounded up to 8): T[g][j] = head_mix[h0 + j][g].
template <int KT, int VDMAX>
__global__ void __launch_bounds__(MT, 1) attn_mix_prefill_mma_kernel(PrefillArgs a, MixCut cut, int subs) {
  extern __shared__ __align__(16) unsigned char smraw[];
  pdl_launch_dependents();
  pdl_wait();
  constexpr int SR = KT + 8;
  const int nh = a.nh, hd = a.hd, vd = a.vd > 0 ? a.vd : a.hd, G = nh / a.nkv;
  const int BQ = 16 * cut.qt, hc8 = (cut.hc + 7) & ~7;
  const int rsk = hd * 2 + 16, rsv = vd * 2 + 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const uint32_t rank = cluster_rank();
  const int h0 = (int)rank * cut.hc, hn = max(0, min(cut.hc, nh - h0));
  const int kv0 = hn > 0 ? h0 / G : 0, kvn = hn > 0 ? (h0 + hn - 1) / G - kv0 + 1 : 0;
  unsigned char* Qs = smraw;
  unsigned char* Ks = Qs + (size_t)cut.hc * BQ * rsk;
  unsigned char* Vs = Ks + (size_t)cut.kvn * KT * rsk;
  float* S = reinterpret_cast<float*>(Vs + (size_t)cut.kvn * KT * rsv);
  float* T = S + (size_t)nh * BQ * SR;
  const int tile_id = (int)blockIdx.y / subs;
  const int b = a.tiles[2 * tile_id], q_off = a.tiles[2 * tile_id + 1] + ((int)blockIdx.y % subs) * BQ;
  const int tok0 = a.cu_tokens[b], t_b = a.cu_tokens[b + 1] - tok0;
  if (q_off >= t_b) return;                       // the same for every block of the cluster
  const int nq = min(BQ, t_b - q_off), lb = a.len_before[b], slot = a.slots[b];
  const int pos0 = lb + q_off, k_end = pos0 + nq;
  const int k_begin = mask_first(pos0, a.window, a.chunked) / KT * KT;
  const int n_tiles = (k_end - k_begin + KT - 1) / KT;
  const bf16 *qg = (const bf16*)a.q, *kn = (const bf16*)a.k_new, *vn = (const bf16*)a.v_new;
  const bf16 *kp = (const bf16*)a.k_pages, *vp = (const bf16*)a.v_pages;

  // rows of a key tile of the block's key/value heads; a tile's old positions lie in one page (KT divides the page)
  // (a thread copies 16-byte piece `ch` of rows r0, r0 + step, ...: no division in the loop)
  const int k_cpr = hd / 8, v_cpr = vd / 8;
  const int k_ch = tid % k_cpr, k_r0 = tid / k_cpr, k_step = MT / k_cpr, v_ch = tid % v_cpr, v_r0 = tid / v_cpr, v_step = MT / v_cpr;
  auto load = [&](int tile, const bf16* fresh_base, const bf16* page_base, int d, unsigned char* dst, int rs, int ch, int r0, int step) {
    const int kt = k_begin + tile * KT;
    const bf16* fresh = fresh_base + ((long long)(tok0 + kt - lb) * a.nkv + kv0) * d + ch * 8;
    const bf16* old = kt < lb ? page_base + kv_row(a.page_table, a.table_width, a.ring_pages, slot, kt, kv0, a.nkv) * d + ch * 8 : nullptr;
    const uint32_t to = smem_u32(dst) + ch * 16;
    if (r0 < step) {
      for (int r = r0; r < kvn * KT; r += step) {
        const int row = r % KT, kv = r / KT, pos = kt + row;
        const bool valid = pos < k_end;
        const bf16* src = pos >= lb ? fresh + (long long)(row * a.nkv + kv) * d : old + (kv * LLG_PAGE + row) * d;
        cp_async16(to + r * rs, valid ? src : fresh_base, valid);
      }
    }
    cp_async_commit();
  };
  for (int idx = tid; idx < hn * BQ * (hd / 8); idx += MT) {
    const int ch = idx % (hd / 8), r = idx / (hd / 8), row = r % BQ, h = r / BQ;
    const bool valid = row < nq;
    cp_async16(smem_u32(Qs + (size_t)r * rsk + ch * 16), qg + ((long long)(tok0 + q_off + (valid ? row : 0)) * nh + h0 + h) * hd + ch * 8, valid);
  }
  load(0, kn, kp, hd, Ks, rsk, k_ch, k_r0, k_step);                   // (one group with the queries)
  for (int idx = tid; idx < nh * hc8; idx += MT) {
    const int j = idx % hc8, gg = idx / hc8;
    T[idx] = j >= hn ? 0.f : a.head_mix ? a.head_mix[(h0 + j) * nh + gg] : (gg == h0 + j ? 1.f : 0.f);
  }
  const int hl = warp % cut.hc, sub = warp / cut.hc;          // this warp's head and 16 queries
  const bool working = sub < cut.qt && hl < hn;
  const int kvl = working ? (h0 + hl) / G - kv0 : 0;
  float o[VDMAX / 8][4];
#pragma unroll
  for (int j = 0; j < VDMAX / 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const float two_over_cap = a.softcap > 0.f ? 2.0f / a.softcap : 0.f;
  const int qpos0 = pos0 + sub * 16 + g;
  const uint32_t s_base = smem_u32(S);
  // pairs of neighbouring positions in a tile (a power of two: qt is 1 or 2), and the mixture's items, at most one a thread
  const int pairs = BQ * (KT / 2), pairs_log2 = 31 - __clz(pairs), items = pairs * (hc8 / 8);
  cluster_arrive();
  for (int tile = 0; tile < n_tiles; ++tile) {
    const int kt = k_begin + tile * KT;
    cp_async_wait<0>();
    __syncthreads();                              // keys are here; every warp is done with the last tile's values
    load(tile, vn, vp, vd, Vs, rsv, v_ch, v_r0, v_step);
    // this warp's scores: 16 queries x KT keys of its head
    float s[KT / 8][4];
    if (working) {
#pragma unroll
      for (int j = 0; j < KT / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
      const uint32_t q_addr = smem_u32(Qs + (size_t)(hl * BQ + sub * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * rsk) + (lane >> 4) * 16;
      const uint32_t k_addr = smem_u32(Ks + (size_t)(kvl * KT + (lane & 7) + (lane >> 4) * 8) * rsk) + ((lane >> 3) & 1) * 16;
#pragma unroll 2
      for (int ks = 0; ks < hd / 16; ++ks) {
        uint32_t qf[4];
        ldmatrix_x4(qf, q_addr + ks * 32);
#pragma unroll
        for (int jp = 0; jp < KT / 16; ++jp) {
          uint32_t kb[4];
          ldmatrix_x4(kb, k_addr + jp * 16 * rsk + ks * 32);
          mma_16816(s[2 * jp], qf, kb[0], kb[1]);
          mma_16816(s[2 * jp + 1], qf, kb[2], kb[3]);
        }
      }
#pragma unroll
      for (int j = 0; j < KT / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[j][e] = capped(s[j][e] * a.scale, a.softcap, two_over_cap);
    }
    cluster_wait();                               // every block has read the last tile's scores
    if (working) {
      const uint32_t at = s_base + (uint32_t)(((h0 + hl) * BQ + sub * 16 + g) * SR + 2 * t) * 4;
      for (uint32_t r = 0; r < (uint32_t)cut.c; ++r) {
        const uint32_t dst = cut.c > 1 ? cluster_addr(at, r) : 0;
#pragma unroll
        for (int j = 0; j < KT / 8; ++j) {
          if (cut.c > 1) {
            cluster_store2(dst + j * 32, s[j][0], s[j][1]);
            cluster_store2(dst + 8 * SR * 4 + j * 32, s[j][2], s[j][3]);
          } else {
            float* p = S + ((h0 + hl) * BQ + sub * 16 + g) * SR + 2 * t + j * 8;
            *reinterpret_cast<float2*>(p) = make_float2(s[j][0], s[j][1]);
            *reinterpret_cast<float2*>(p + 8 * SR) = make_float2(s[j][2], s[j][3]);
          }
        }
      }
    }
    cluster_arrive();
    cluster_wait();                               // all heads' scores are here; the keys may be replaced
    if (tile + 1 < n_tiles) load(tile + 1, kn, kp, hd, Ks, rsk, k_ch, k_r0, k_step);
    else cp_async_commit();
    // the mixture: an item is two neighbouring positions for eight of the block's heads
    float mx[8][2];
    const bool mixing = tid < items;
    float* sp = S + ((tid & (pairs - 1)) / (KT / 2)) * SR + 2 * (tid % (KT / 2));
    const int j0 = (tid >> pairs_log2) * 8;
    if (mixing) {
#pragma unroll
      for (int j = 0; j < 8; ++j) mx[j][0] = mx[j][1] = 0.f;
      const float* tp = T + j0;
#pragma unroll 4
      for (int gg = 0; gg < nh; ++gg) {
        const float2 v = *reinterpret_cast<const float2*>(sp + gg * BQ * SR);
        const float4 t0 = *reinterpret_cast<const float4*>(tp + gg * hc8), t1 = *reinterpret_cast<const float4*>(tp + gg * hc8 + 4);
        const float tt[8] = {t0.x, t0.y, t0.z, t0.w, t1.x, t1.y, t1.z, t1.w};
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          mx[j][0] = fmaf(tt[j], v.x, mx[j][0]);
          mx[j][1] = fmaf(tt[j], v.y, mx[j][1]);
        }
      }
    }
    __syncthreads();                              // every thread has read all heads' scores: the mixed ones take their place
    if (mixing) {
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (j0 + j < hn) *reinterpret_cast<float2*>(sp + (j0 + j) * BQ * SR) = make_float2(mx[j][0], mx[j][1]);
    }
    cp_async_wait<1>();                           // the values are here (the next keys may still be on their way)
    __syncthreads();
    if (working) {
      const float* p = S + (hl * BQ + sub * 16 + g) * SR + 2 * t;
#pragma unroll
      for (int j = 0; j < KT / 8; ++j) {
        const float2 u = *reinterpret_cast<const float2*>(p + j * 8), v = *reinterpret_cast<const float2*>(p + 8 * SR + j * 8);
        s[j][0] = u.x; s[j][1] = u.y; s[j][2] = v.x; s[j][3] = v.y;
      }
    }
    cluster_arrive();                             // this block no longer needs the scores
    if (!working) continue;
    if (kt + KT - 1 > pos0 + sub * 16 || (a.window > 0 && kt < mask_first(pos0 + sub * 16 + 15, a.window, a.chunked))) {
#pragma unroll
      for (int j = 0; j < KT / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int key = kt + j * 8 + 2 * t + (e & 1), qp = qpos0 + (e >> 1) * 8;
          if (key > qp || key < mask_first(qp, a.window, a.chunked)) s[j][e] = -INFINITY;
        }
    }
    // the running maximum is a whole number of log2 units, as in attention_mma.cu: rescaling is exact
    float top[2] = {-INFINITY, -INFINITY}, corr[2];
#pragma unroll
    for (int j = 0; j < KT / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) top[e >> 1] = fmaxf(top[e >> 1], s[j][e]);
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      top[r] = fmaxf(top[r], __shfl_xor_sync(0xffffffffu, top[r], 1));
      top[r] = fmaxf(top[r], __shfl_xor_sync(0xffffffffu, top[r], 2));
      const float m_new = fmaxf(m[r], ceilf(top[r] * LOG2E));
      corr[r] = m_new == -INFINITY ? 1.f : pow2_whole(m[r] - m_new);
      m[r] = m_new;
      l[r] *= corr[r];
    }
    const float ms[2] = {m[0] == -INFINITY ? 0.f : m[0], m[1] == -INFINITY ? 0.f : m[1]};
#pragma unroll
    for (int j = 0; j < KT / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float p = fast_exp2(fmaf(s[j][e], LOG2E, -ms[e >> 1]));
        s[j][e] = p;
        l[e >> 1] += p;
      }
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
      for (int j = 0; j < VDMAX / 8; ++j) {
        o[j][0] *= corr[0]; o[j][1] *= corr[0]; o[j][2] *= corr[1]; o[j][3] *= corr[1];
      }
    }
    const uint32_t v_addr = smem_u32(Vs + (size_t)(kvl * KT + (lane & 7) + ((lane >> 3) & 1) * 8) * rsv) + (lane >> 4) * 16;
#pragma unroll
    for (int kk = 0; kk < KT / 16; ++kk) {
      const uint32_t pa[4] = {pack_bf16(s[2 * kk][0], s[2 * kk][1]), pack_bf16(s[2 * kk][2], s[2 * kk][3]),
                              pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]), pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
      for (int jp = 0; jp < VDMAX / 16; ++jp) {
        if (jp * 16 < vd) {
          uint32_t vb[4];
          ldmatrix_x4_trans(vb, v_addr + kk * 16 * rsv + jp * 32);
          mma_16816(o[2 * jp], pa, vb[0], vb[1]);
          mma_16816(o[2 * jp + 1], pa, vb[2], vb[3]);
        }
      }
    }
  }
  cluster_wait();                                 // no block leaves while another may still write into its shared memory
  if (!working) return;
  bf16* out = (bf16*)a.out;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const int row = sub * 16 + g + r * 8, h = h0 + hl;
    if (row >= nq) continue;
    float lr = l[r];
    if (a.has_sink) lr += fast_exp2((a.sinks ? a.sinks[h] : a.sink_score) * LOG2E - m[r]);
    float inv = lr > 0.f ? 1.0f / lr : 0.f;
    if (a.gate) inv *= a.gate[(long long)(tok0 + q_off + row) * nh + h];
    bf16* dst = out + ((long long)(tok0 + q_off + row) * nh + h) * vd;
#pragma unroll
    for (int j = 0; j < VDMAX / 8; ++j)
      if (j * 8 < vd) *reinterpret_cast<uint32_t*>(dst + j * 8 + 2 * t) = pack_bf16(o[j][2 * r] * inv, o[j][2 * r + 1] * inv);
  }
}

// ---- one new token per sequence ------------------------------------------------------------------

constexpr int DK = 16;                  // keys per tile
constexpr int DS = DK + 8;              // floats per row of scores
constexpr int MAX_STAGES = 6;           // tiles of keys and values in shared memory at most
constexpr int PR = DK * 2 + 16;         // bytes per row of weights
constexpr int MAX_ACC = 8;              // 16-row x 16-column pieces of the outputs that a warp may own
constexpr int MAX_ROWS = 4;             // heads whose softmax half a warp may own

// Shared memory: Q [nh][rsk], `stages` times K [nkv][DK][rsk] and V [nkv][DK][rsv], P [nh][PR] bytes, then floats: scores
// [nh][DS], corr [nh], the mixture [nh][nh].  A tile's keys and values arrive together, stages - 1 tiles ahead.
__global__ void __launch_bounds__(MT, 1) attn_mix_decode_mma_kernel(DecodeArgs a, int stages) {
  extern __shared__ __align__(16) unsigned char smraw[];
  pdl_launch_dependents();
  pdl_wait();
  const int nh = a.nh, nkv = a.nkv, hd = a.hd, vd = a.vd > 0 ? a.vd : a.hd, G = nh / nkv, RC = (G + 15) / 16;
  const int rsk = hd * 2 + 16, rsv = vd * 2 + 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int split = blockIdx.x, b = blockIdx.y;
  unsigned char* Qs = smraw;
  unsigned char* Ks = Qs + (size_t)nh * rsk;
  const int k_bytes = nkv * DK * rsk, stage_bytes = k_bytes + nkv * DK * rsv;
  unsigned char* Ps = Ks + (size_t)stages * stage_bytes;
  float* S = reinterpret_cast<float*>(Ps + (size_t)nh * PR);
  float* corr = S + nh * DS;
  float* T = corr + nh;
  const int len = a.len_before[b] + 1, slot = a.slots[b];
  const int lo = mask_first(len - 1, a.window, a.chunked);
  const int t0 = lo / DK, t_end = (len + DK - 1) / DK;
  const int per = (t_end - t0 + a.n_splits - 1) / a.n_splits;
  const int my0 = min(t_end, t0 + split * per), my1 = min(t_end, my0 + per);
  const bf16 *qg = (const bf16*)a.q + (long long)b * nh * hd, *kp = (const bf16*)a.k_pages, *vp = (const bf16*)a.v_pages;
  const int k_cpr = hd / 8, v_cpr = vd / 8;
  const int k_ch = tid % k_cpr, k_r0 = tid / k_cpr, k_step = MT / k_cpr, v_ch = tid % v_cpr, v_r0 = tid / v_cpr, v_step = MT / v_cpr;
  const uint32_t k_to = smem_u32(Ks) + k_ch * 16, v_to = smem_u32(Ks) + k_bytes + v_ch * 16;
  const bool k_copies = k_r0 < k_step, v_copies = v_r0 < v_step;
  // the page of a tile is looked up one tile ahead of its copies
  auto page_of = [&](int tile) {
    return tile < my1 ? a.page_table[(long long)slot * a.table_width + (tile * DK / LLG_PAGE) % a.ring_pages] : 0;
  };
  int page = page_of(my0);
  auto load = [&](int tile, int stage) {
    if (tile < my1) {
      const int pos0 = tile * DK;
      const long long base = (long long)page * nkv * LLG_PAGE + pos0 % LLG_PAGE;
      page = page_of(tile + 1);
      if (k_copies) {
        const bf16* src = kp + base * hd + k_ch * 8;
        for (int r = k_r0; r < nkv * DK; r += k_step) {
          const bool valid = pos0 + r % DK < len;
          cp_async16(k_to + stage * stage_bytes + r * rsk, valid ? src + (long long)(r / DK * LLG_PAGE + r % DK) * hd : kp, valid);
        }
      }
      if (v_copies) {
        const bf16* src = vp + base * vd + v_ch * 8;
        for (int r = v_r0; r < nkv * DK; r += v_step) {
          const bool valid = pos0 + r % DK < len;
          cp_async16(v_to + stage * stage_bytes + r * rsv, valid ? src + (long long)(r / DK * LLG_PAGE + r % DK) * vd : vp, valid);
        }
      }
    }
    cp_async_commit();
  };
  for (int idx = tid; idx < nh * (hd / 8); idx += MT) {
    const int ch = idx % (hd / 8), h = idx / (hd / 8);
    cp_async16(smem_u32(Qs + (size_t)h * rsk + ch * 16), qg + (long long)h * hd + ch * 8, true);
  }
  for (int st = 0; st < stages - 1; ++st) load(my0 + st, st);      // (the queries belong to the first group)
  for (int idx = tid; idx < nh * nh; idx += MT) T[idx] = a.head_mix ? a.head_mix[idx] : (idx / nh == idx % nh ? 1.f : 0.f);
  const int v16 = vd / 16, acc_items = nkv * RC * v16, qk_items = nkv * RC * (DK / 16);
  float o[MAX_ACC][2][4];
#pragma unroll
  for (int i = 0; i < MAX_ACC; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][0][e] = o[i][1][e] = 0.f;
  float m[MAX_ROWS], l[MAX_ROWS];
#pragma unroll
  for (int i = 0; i < MAX_ROWS; ++i) {
    m[i] = -INFINITY;
    l[i] = 0.f;
  }
  const float two_over_cap = a.softcap > 0.f ? 2.0f / a.softcap : 0.f;
  const int frag_row = (lane & 7) + ((lane >> 3) & 1) * 8;
  // this warp's pieces of the outputs: shared-memory offsets of their weights' and values' rows, first head
  int p_off[MAX_ACC], v_off[MAX_ACC], c_off[MAX_ACC];
#pragma unroll
  for (int i = 0; i < MAX_ACC; ++i) {
    const int it = min(warp + i * MW, acc_items - 1), vc = it % v16, u = it / v16, row0 = u / RC * G + u % RC * 16;
    p_off[i] = min(row0 + frag_row, nh - 1) * PR + (lane >> 4) * 16;
    v_off[i] = (u / RC * DK + frag_row) * rsv + (lane >> 4) * 16 + vc * 32;
    c_off[i] = min(row0 + g, nh - 1) | min(row0 + g + 8, nh - 1) << 16;
  }
  const uint32_t ps_at = smem_u32(Ps);
  int stage = 0;
  for (int tile = my0; tile < my1; ++tile) {
    if (stages == 2) cp_async_wait<0>();
    else if (stages == 3) cp_async_wait<1>();
    else if (stages == 4) cp_async_wait<2>();
    else if (stages == 5) cp_async_wait<3>();
    else cp_async_wait<4>();
    __syncthreads();                              // the tile is here; the tile before last is no longer read
    load(tile + stages - 1, stage == 0 ? stages - 1 : stage - 1);
    const uint32_t k_at = smem_u32(Ks) + stage * stage_bytes, v_at = k_at + k_bytes;
    stage = stage + 1 == stages ? 0 : stage + 1;
    for (int it = warp; it < qk_items; it += MW) {
      const int kh = it % (DK / 16), u = it / (DK / 16), rc = RC == 1 ? 0 : u % RC, kv = RC == 1 ? u : u / RC;
      const int row0 = kv * G + rc * 16;
      const uint32_t q_addr = smem_u32(Qs + (size_t)min(row0 + frag_row, nh - 1) * rsk) + (lane >> 4) * 16;
      const uint32_t k_addr = k_at + (kv * DK + kh * 16 + (lane & 7) + (lane >> 4) * 8) * rsk + ((lane >> 3) & 1) * 16;
      float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll 4
      for (int ks = 0; ks < hd / 16; ++ks) {
        uint32_t qf[4], kb[4];
        ldmatrix_x4(qf, q_addr + ks * 32);
        ldmatrix_x4(kb, k_addr + ks * 32);
        mma_16816(s[0], qf, kb[0], kb[1]);
        mma_16816(s[1], qf, kb[2], kb[3]);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r)
          if (rc * 16 + g + r * 8 < G)
            *reinterpret_cast<float2*>(S + (row0 + g + r * 8) * DS + kh * 16 + j * 8 + 2 * t) =
                make_float2(capped(s[j][2 * r] * a.scale, a.softcap, two_over_cap), capped(s[j][2 * r + 1] * a.scale, a.softcap, two_over_cap));
    }
    __syncthreads();
    // mixture and softmax: half a warp per head, a lane per key
    const int key = lane & 15, pos = tile * DK + key;
    const bool valid = pos < len && pos >= lo;
#pragma unroll
    for (int i = 0; i < MAX_ROWS; ++i) {
      const int h = 2 * warp + (lane >> 4) + i * 2 * MW;
      if (2 * warp + i * 2 * MW >= nh) break;
      const bool mine = h < nh;
      const float* tr = T + (mine ? h : 0) * nh;
      float s4[4] = {0.f, 0.f, 0.f, 0.f};
      int gg = 0;
      for (; gg + 4 <= nh; gg += 4) {
#pragma unroll
        for (int x = 0; x < 4; ++x) s4[x] = fmaf(tr[gg + x], S[(gg + x) * DS + key], s4[x]);
      }
      for (; gg < nh; ++gg) s4[0] = fmaf(tr[gg], S[gg * DS + key], s4[0]);
      float s = (s4[0] + s4[1]) + (s4[2] + s4[3]);
      if (!valid) s = -INFINITY;
      float mx = s;
#pragma unroll
      for (int x = 8; x > 0; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
      const float m_new = fmaxf(m[i], ceilf(mx * LOG2E));
      const float c = m_new == -INFINITY ? 1.f : pow2_whole(m[i] - m_new);
      const float p = m_new == -INFINITY ? 0.f : fast_exp2(fmaf(s, LOG2E, -m_new));
      m[i] = m_new;
      l[i] = l[i] * c + p;                        // this lane's share of the sum
      if (mine) {
        *reinterpret_cast<bf16*>(Ps + (size_t)h * PR + key * 2) = __float2bfloat16_rn(p);
        if (key == 0) corr[h] = c;
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MAX_ACC; ++i) {
      const int it = warp + i * MW;
      if (it >= acc_items) break;
      const float c0 = corr[c_off[i] & 0xffff], c1 = corr[c_off[i] >> 16];
      const uint32_t p_addr = ps_at + p_off[i], v_addr = v_at + v_off[i];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        o[i][j][0] *= c0; o[i][j][1] *= c0; o[i][j][2] *= c1; o[i][j][3] *= c1;
      }
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
        uint32_t pa[4], vb[4];
        ldmatrix_x4(pa, p_addr + kk * 32);
        ldmatrix_x4_trans(vb, v_addr + kk * 16 * rsv);
        mma_16816(o[i][0], pa, vb[0], vb[1]);
        mma_16816(o[i][1], pa, vb[2], vb[3]);
      }
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int i = 0; i < MAX_ACC; ++i) {
    const int it = warp + i * MW;
    if (it >= acc_items) break;
    const int vc = it % v16, u = it / v16, rc = u % RC, kv = u / RC;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      if (rc * 16 + g + r * 8 >= G) continue;
      const int h = kv * G + rc * 16 + g + r * 8;
      float* dst = a.part_o + (((long long)b * nh + h) * a.n_splits + split) * vd + vc * 16 + 2 * t;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        dst[j * 8] = o[i][j][2 * r];
        dst[j * 8 + 1] = o[i][j][2 * r + 1];
      }
    }
  }
#pragma unroll
  for (int i = 0; i < MAX_ROWS; ++i) {
    const int h = 2 * warp + (lane >> 4) + i * 2 * MW;
    if (2 * warp + i * 2 * MW >= nh) break;
    float sum = l[i];
#pragma unroll
    for (int x = 8; x > 0; x >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, x);
    if ((lane & 15) == 0 && h < nh) {
      float* ml = a.part_ml + (((long long)b * nh + h) * a.n_splits + split) * 2;
      ml[0] = m[i] == -INFINITY ? -INFINITY : m[i] * 0.6931471805599453f;      // natural units
      ml[1] = sum;
    }
  }
}

constexpr size_t SMEM_MAX = 227 * 1024;

size_t prefill_smem(int nh, int hd, int vd, const MixCut& c) {
  const size_t bq = 16 * c.qt, rsk = 2 * hd + 16, rsv = 2 * vd + 16, hc8 = (c.hc + 7) & ~7;
  return (size_t)c.hc * bq * rsk + (size_t)c.kvn * c.kt * (rsk + rsv) + ((size_t)nh * bq * mix_score_stride(c.kt) + (size_t)nh * hc8) * sizeof(float);
}

// The cut of a prompt step for these sizes: as few blocks per cluster and as many keys per tile as shared memory allows.
bool plan_prefill(int nh, int nkv, int hd, int vd, MixCut* out) {
  const int G = nh / nkv;
  for (int c = (nh + MW - 1) / MW; c <= 8; ++c) {
    for (int kt = 32; kt >= 16; kt -= 16) {
      MixCut p;
      p.c = c;
      p.hc = (nh + c - 1) / c;
      p.qt = p.hc <= 8 ? 2 : 1;                   // at most MT items of the mixture
      p.kt = kt;
      p.kvn = 0;                                  // the most key/value heads that a block's heads reach
      for (int h0 = 0; h0 < nh; h0 += p.hc) p.kvn = max(p.kvn, (min(h0 + p.hc, nh) - 1) / G - h0 / G + 1);
      p.smem = prefill_smem(nh, hd, vd, p);
      if (p.smem <= SMEM_MAX) {
        *out = p;
        return true;
      }
    }
  }
  return false;
}

size_t decode_smem(int nh, int nkv, int hd, int vd, int stages) {
  const size_t rsk = 2 * hd + 16, rsv = 2 * vd + 16;
  return (size_t)nh * rsk + (size_t)stages * nkv * DK * (rsk + rsv) + (size_t)nh * PR + ((size_t)nh * DS + nh + (size_t)nh * nh) * sizeof(float);
}

bool head_sizes_ok(int nh, int nkv, int hd, int vd) {
  return nh > 0 && nkv > 0 && nh % nkv == 0 && nh <= 2 * MW * MAX_ROWS && hd >= 16 && hd <= 128 && hd % 16 == 0 && vd >= 16 && vd <= 128 && vd % 16 == 0;
}

}  // namespace

// 1 when the kernels of this file take these sizes.
LLG_API int llg_attn_mix_prefill_mma_supported(int nh, int nkv, int hd, int vd) {
  MixCut p;
  return head_sizes_ok(nh, nkv, hd, vd) && plan_prefill(nh, nkv, hd, vd, &p);
}
LLG_API int llg_attn_mix_decode_mma_supported(int nh, int nkv, int hd, int vd) {
  if (!head_sizes_ok(nh, nkv, hd, vd)) return 0;
  const int G = nh / nkv;
  return nkv * ((G + 15) / 16) * (vd / 16) <= MW * MAX_ACC && decode_smem(nh, nkv, hd, vd, 2) <= SMEM_MAX;
}

// tile_queries: queries per entry of `tiles`, a multiple of 64.
LLG_API int llg_attn_mix_prefill_mma(const PrefillArgs* args, int tile_queries, cudaStream_t stream) {
  const PrefillArgs& a = *args;
  const int vd = a.vd > 0 ? a.vd : a.hd;
  MixCut cut;
  LLG_REQUIRE(head_sizes_ok(a.nh, a.nkv, a.hd, vd) && plan_prefill(a.nh, a.nkv, a.hd, vd, &cut),
              "attn_mix_prefill_mma: %d heads (%d) of %d and %d elements", a.nh, a.nkv, a.hd, vd);
  LLG_REQUIRE(a.scale > 0.f && a.softcap >= 0.f, "attn_mix_prefill_mma: scale %g, cap %g", a.scale, a.softcap);
  LLG_REQUIRE(a.window >= 0 && a.ring_pages > 0 && a.table_width >= a.ring_pages, "attn_mix_prefill_mma: bad cache geometry");
  LLG_REQUIRE(tile_queries > 0 && tile_queries % 64 == 0, "attn_mix_prefill_mma: tiles of %d queries", tile_queries);
  if (a.n_tiles <= 0) return 0;
  const int subs = tile_queries / (16 * cut.qt);
  LLG_REQUIRE((long long)a.n_tiles * subs <= 65535, "attn_mix_prefill_mma: %d tiles of %d queries in one step", a.n_tiles, tile_queries);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(cut.c, (unsigned)(a.n_tiles * subs));
  cfg.blockDim = dim3(MT);
  cfg.dynamicSmemBytes = cut.smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cut.c;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = llg_pdl_enabled() ? 2 : 1;
#define GO(KT, VD)                                                                                                     \
  do {                                                                                                                 \
    auto k = attn_mix_prefill_mma_kernel<KT, VD>;                                                                      \
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)cut.smem);               \
    if (e == cudaSuccess) e = cudaLaunchKernelEx(&cfg, k, a, cut, subs);                                               \
    if (e != cudaSuccess) return llg_fail("attn_mix_prefill_mma: %s", cudaGetErrorString(e));                          \
    return llg_check_launch("attn_mix_prefill_mma");                                                                   \
  } while (0)
  if (cut.kt == 32) {
    if (vd <= 64) GO(32, 64);
    GO(32, 128);
  }
  if (vd <= 64) GO(16, 64);
  GO(16, 128);
#undef GO
}

LLG_API int llg_attn_mix_decode_mma(const DecodeArgs* args, void* out, cudaStream_t stream) {
  const DecodeArgs& a = *args;
  const int vd = a.vd > 0 ? a.vd : a.hd;
  LLG_REQUIRE(llg_attn_mix_decode_mma_supported(a.nh, a.nkv, a.hd, vd), "attn_mix_decode_mma: %d heads (%d) of %d and %d elements", a.nh,
              a.nkv, a.hd, vd);
  LLG_REQUIRE(a.scale > 0.f && a.softcap >= 0.f, "attn_mix_decode_mma: scale %g, cap %g", a.scale, a.softcap);
  LLG_REQUIRE(a.n_splits >= 1 && a.n_splits <= 65535 && a.n_seqs <= 65535, "attn_mix_decode_mma: grid too large");
  LLG_REQUIRE(a.window >= 0 && a.ring_pages > 0 && a.table_width >= a.ring_pages, "attn_mix_decode_mma: bad cache geometry");
  if (a.n_seqs <= 0) return 0;
  int stages = 2;
  while (stages < MAX_STAGES && decode_smem(a.nh, a.nkv, a.hd, vd, stages + 1) <= SMEM_MAX) ++stages;
  const size_t smem = decode_smem(a.nh, a.nkv, a.hd, vd, stages);
  cudaError_t e = cudaFuncSetAttribute(attn_mix_decode_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return llg_fail("attn_mix_decode_mma: shared memory %zu: %s", smem, cudaGetErrorString(e));
  llg_launch(attn_mix_decode_mma_kernel, dim3(a.n_splits, a.n_seqs), dim3(MT), smem, stream, a, stages);
  attn_decode_reduce_kernel<bf16><<<dim3(a.nh, a.n_seqs), 64, 0, stream>>>(a.part_o, a.part_ml, (bf16*)out, a.nh, vd, a.n_splits, a.has_sink,
                                                                        a.sink_score, a.gate, a.sinks);
  return llg_check_launch("attn_mix_decode_mma");
}
