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
//   attn_mix_decode_mma  : one new token per sequence; scores, mixture with weights, and values by a kernel each (the partial
//                          results of a sequence's key splits are joined by attn_decode_reduce).
//
// In prompt steps shared-memory rows of bfloat16 are padded by 16 bytes (conflict-free ldmatrix), rows of scores by 8 floats.
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
//
// Three kernels that each stream what they read once, over all the GPU's blocks: the scores of every head (keys read straight
// into operand registers, a warp per 16 keys of one key/value head), the mixture with the softmax's weights per chunk of
// CHUNK keys, and the weighted values (read straight into operand registers again).  Between them lie, per sequence, the
// scores [key][nh] in float32, the weights [nh][key] in bfloat16, and per (head, chunk) the maximum and the sum.  Keys are
// counted from the first page that the query sees.
//
// The order of the elements inside a product over the head's elements is free, and so is the order of an output's columns.
// Both are chosen so that a lane's operands are 16 neighbouring bytes of a row: for the scores lane (g, t) takes elements
// 32 c + 8 t .. + 7 of keys g and g + 8 as the operands of two products; for the values lane (g, t) takes elements
// 64 c + 8 g .. + 7 of keys 2t, 2t + 1, 2t + 8, 2t + 9, and product j of eight uses element j of each.

constexpr int CHUNK = LLG_PAGE;         // keys per chunk of the softmax (one page)

struct MixScratch {
  float* scores;                        // [n_seqs][keys][nh]
  bf16* weights;                        // [n_seqs][nh][keys]
  float* chunks;                        // [n_seqs][nh][keys / CHUNK][2]: maximum (whole log2 units), sum
  int keys;                             // most keys of a sequence, whole chunks
};

__device__ __forceinline__ int first_page_key(const DecodeArgs& a, int len) { return mask_first(len - 1, a.window, a.chunked) / LLG_PAGE * LLG_PAGE; }
__device__ __forceinline__ int page_at(const DecodeArgs& a, int slot, int pos) {
  return a.page_table[(long long)slot * a.table_width + (pos / LLG_PAGE) % a.ring_pages];
}

// HD32: the head's elements in steps of 32, at most (a remainder of 16 is one product more)
template <int HD32>
__global__ void __launch_bounds__(128, 4) mix_scores_kernel(DecodeArgs a, MixScratch w) {
  pdl_launch_dependents();
  const int nh = a.nh, nkv = a.nkv, hd = a.hd, G = nh / nkv;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int kv = blockIdx.y, b = blockIdx.z;
  pdl_wait();
  const int len = a.len_before[b] + 1, base = first_page_key(a, len);
  const int n_chunks = (len - base + CHUNK - 1) / CHUNK, per = (n_chunks + gridDim.x - 1) / gridDim.x;
  const int c0 = blockIdx.x * per, c1 = min(n_chunks, c0 + per);
  if (c0 >= c1) return;
  const int slot = a.slots[b], steps = hd / 32, tail = hd % 32;
  const float two_over_cap = a.softcap > 0.f ? 2.0f / a.softcap : 0.f;
  const bf16* q = (const bf16*)a.q + ((long long)b * nh + kv * G) * hd;
  struct Keys {
    uint4 lo[HD32], hi[HD32];
    uint2 t_lo, t_hi;
  };
  auto fetch = [&](Keys& k, int page) {
    const bf16* row = (const bf16*)a.k_pages + (((long long)page * nkv + kv) * LLG_PAGE + warp * 16 + g) * hd;
#pragma unroll
    for (int c = 0; c < HD32; ++c)
      if (c < steps) {
        k.lo[c] = *reinterpret_cast<const uint4*>(row + c * 32 + t * 8);
        k.hi[c] = *reinterpret_cast<const uint4*>(row + 8 * hd + c * 32 + t * 8);
      }
    if (tail) {
      k.t_lo = *reinterpret_cast<const uint2*>(row + steps * 32 + t * 4);
      k.t_hi = *reinterpret_cast<const uint2*>(row + 8 * hd + steps * 32 + t * 4);
    }
  };
  auto score = [&](const Keys& k, int chunk) {
    float* dst = w.scores + ((long long)b * w.keys + chunk * CHUNK + warp * 16 + g) * nh + kv * G;
    for (int g0 = 0; g0 < G; g0 += 8) {
      const bf16* qr = q + (long long)min(g0 + g, G - 1) * hd;        // column g of the product: head g0 + g
      float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int c = 0; c < HD32; ++c)
        if (c < steps) {
          const uint4 qf = *reinterpret_cast<const uint4*>(qr + c * 32 + t * 8);
          const uint32_t a0[4] = {k.lo[c].x, k.hi[c].x, k.lo[c].y, k.hi[c].y}, a1[4] = {k.lo[c].z, k.hi[c].z, k.lo[c].w, k.hi[c].w};
          mma_16816(s0, a0, qf.x, qf.y);
          mma_16816(s1, a1, qf.z, qf.w);
        }
      if (tail) {
        const uint2 qf = *reinterpret_cast<const uint2*>(qr + steps * 32 + t * 4);
        const uint32_t a0[4] = {k.t_lo.x, k.t_hi.x, k.t_lo.y, k.t_hi.y};
        mma_16816(s0, a0, qf.x, qf.y);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {                 // keys g (e < 2) and g + 8, heads g0 + 2t and g0 + 2t + 1
        const int h = g0 + 2 * t + (e & 1);
        if (h < G) dst[(long long)(e >> 1) * 8 * nh + h] = capped((s0[e] + s1[e]) * a.scale, a.softcap, two_over_cap);
      }
    }
  };
  // the next keys are on their way while the products of these run
  Keys ka, kb;
  auto page_of = [&](int c) { return c < c1 ? page_at(a, slot, base + c * CHUNK) : 0; };
  int next = page_of(c0 + 1);
  fetch(ka, page_of(c0));
  for (int c = c0; c < c1; c += 2) {
    if (c + 1 < c1) fetch(kb, next);
    next = page_of(c + 2);
    score(ka, c);
    if (c + 1 >= c1) break;
    if (c + 2 < c1) fetch(ka, next);
    next = page_of(c + 3);
    score(kb, c + 1);
  }
}

// rows of scores and of the mixture in shared memory, in floats: the heads filled up to a multiple of four, and four more
// so that neighbouring rows start in different banks
__host__ __device__ inline int heads_stride(int nh) { return (nh + 3) / 4 * 4 + 4; }

// The mixture and a chunk's softmax: a warp takes four heads at a time, a lane two keys.
__global__ void __launch_bounds__(256) mix_weights_kernel(DecodeArgs a, MixScratch w) {
  extern __shared__ __align__(16) float msm[];
  pdl_launch_dependents();
  const int nh = a.nh, hs = heads_stride(nh), nh4 = (nh + 3) & ~3;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, b = blockIdx.y;
  float* T = msm;                                 // [nh4][hs]
  float* S = T + nh4 * hs;                        // [CHUNK][hs]
  const bool vec = nh % 4 == 0;
  if (vec && a.head_mix) {
    const int q4 = nh / 4, step = 256 / q4, c = threadIdx.x % q4;
    for (int h = threadIdx.x / q4; h < nh && threadIdx.x < step * q4; h += step)
      *reinterpret_cast<float4*>(T + h * hs + c * 4) = *reinterpret_cast<const float4*>(a.head_mix + h * nh + c * 4);
  } else {
    for (int idx = threadIdx.x; idx < nh4 * hs; idx += 256) {
      const int h = idx / hs, gg = idx - h * hs;
      T[idx] = h >= nh || gg >= nh ? 0.f : a.head_mix ? a.head_mix[h * nh + gg] : (h == gg ? 1.f : 0.f);
    }
  }
  pdl_wait();
  const int len = a.len_before[b] + 1, lo = mask_first(len - 1, a.window, a.chunked), base = lo / LLG_PAGE * LLG_PAGE;
  const int r0 = blockIdx.x * CHUNK;
  if (base + r0 >= len) return;
  const float* src = w.scores + ((long long)b * w.keys + r0) * nh;
  if (vec) {
    const int q4 = nh / 4, step = 256 / q4, c = threadIdx.x % q4;
    for (int k = threadIdx.x / q4; k < CHUNK && threadIdx.x < step * q4; k += step)
      *reinterpret_cast<float4*>(S + k * hs + c * 4) =
          base + r0 + k < len ? *reinterpret_cast<const float4*>(src + k * nh + c * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
  } else {
    for (int idx = threadIdx.x; idx < CHUNK * nh; idx += 256) {
      const int k = idx / nh, h = idx - k * nh;
      S[k * hs + h] = base + r0 + k < len ? src[idx] : 0.f;
    }
    for (int idx = threadIdx.x; idx < CHUNK * (hs - nh); idx += 256) S[idx / (hs - nh) * hs + nh + idx % (hs - nh)] = 0.f;
  }
  __syncthreads();
  for (int h0 = warp * 4; h0 < nh; h0 += 32) {
    float acc[4][2] = {};
    for (int gg = 0; gg < nh4; gg += 4) {
      const float4 x = *reinterpret_cast<const float4*>(S + lane * hs + gg), y = *reinterpret_cast<const float4*>(S + (lane + 32) * hs + gg);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float4 m = *reinterpret_cast<const float4*>(T + (h0 + j) * hs + gg);
        acc[j][0] = fmaf(m.x, x.x, acc[j][0]); acc[j][1] = fmaf(m.x, y.x, acc[j][1]);
        acc[j][0] = fmaf(m.y, x.y, acc[j][0]); acc[j][1] = fmaf(m.y, y.y, acc[j][1]);
        acc[j][0] = fmaf(m.z, x.z, acc[j][0]); acc[j][1] = fmaf(m.z, y.z, acc[j][1]);
        acc[j][0] = fmaf(m.w, x.w, acc[j][0]); acc[j][1] = fmaf(m.w, y.w, acc[j][1]);
      }
    }
    const int p0 = base + r0 + lane, p1 = p0 + 32;
    const bool v0 = p0 < len && p0 >= lo, v1 = p1 < len && p1 >= lo;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int h = h0 + j;
      if (h >= nh) break;
      const float top = warp_max(fmaxf(v0 ? acc[j][0] : -INFINITY, v1 ? acc[j][1] : -INFINITY));
      const float m = ceilf(top * LOG2E);         // whole log2 units: rescaling between chunks is exact
      const float e0 = v0 ? fast_exp2(fmaf(acc[j][0], LOG2E, -m)) : 0.f, e1 = v1 ? fast_exp2(fmaf(acc[j][1], LOG2E, -m)) : 0.f;
      const float sum = warp_sum(e0 + e1);
      bf16* dst = w.weights + ((long long)b * nh + h) * w.keys + r0 + lane;
      dst[0] = __float2bfloat16_rn(e0);
      dst[32] = __float2bfloat16_rn(e1);
      if (lane == 0) {
        float* c = w.chunks + (((long long)b * nh + h) * (w.keys / CHUNK) + blockIdx.x) * 2;
        c[0] = m;
        c[1] = sum;
      }
    }
  }
}

// The weighted values: block (split, key/value head, up to 16 of its query heads and 64 of its elements, sequence); the four
// warps take a chunk's four runs of 16 keys, and the next chunk's values are on their way while a chunk's products run.  All partial results are relative to the sequence's largest maximum.
__global__ void __launch_bounds__(128, 4) mix_values_kernel(DecodeArgs a, MixScratch w) {
  pdl_launch_dependents();
  __shared__ float top_of[16], merge[4][16][64 + 4];
  const int nh = a.nh, nkv = a.nkv, vd = a.vd > 0 ? a.vd : a.hd, G = nh / nkv, RC = (G + 15) / 16, NX = (vd + 63) / 64;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int split = blockIdx.x, x = blockIdx.y % NX, u = blockIdx.y / NX, kv = u / RC, h0 = kv * G + u % RC * 16, b = blockIdx.z;
  const int gn = min(16, kv * G + G - h0);        // heads of this block
  pdl_wait();
  const int len = a.len_before[b] + 1, base = first_page_key(a, len), slot = a.slots[b];
  const int n_chunks = (len - base + CHUNK - 1) / CHUNK, all = w.keys / CHUNK;
  const int per = (n_chunks + a.n_splits - 1) / a.n_splits;
  const int c0 = min(n_chunks, split * per), c1 = min(n_chunks, c0 + per);
  const float* ch = w.chunks + ((long long)b * nh + h0) * all * 2;
  // the largest maximum of every head, and this split's share of the sum
  for (int h = warp; h < gn; h += 4) {
    float m = -INFINITY, l = 0.f;
    for (int c = lane; c < n_chunks; c += 32) m = fmaxf(m, ch[((long long)h * all + c) * 2]);
    m = warp_max(m);
    for (int c = c0 + lane; c < c1; c += 32) l += pow2_whole(ch[((long long)h * all + c) * 2] - m) * ch[((long long)h * all + c) * 2 + 1];
    l = warp_sum(l);
    if (lane == 0) top_of[h] = m;
    if (lane == 0 && x == 0) {
      float* ml = a.part_ml + (((long long)b * nh + h0 + h) * a.n_splits + split) * 2;
      ml[0] = c0 < c1 ? m * 0.6931471805599453f : -INFINITY;          // natural units
      ml[1] = l;
    }
  }
  __syncthreads();
  const float m0 = top_of[min(g, gn - 1)], m1 = top_of[min(g + 8, gn - 1)];
  const bf16* p0 = w.weights + ((long long)b * nh + h0 + min(g, gn - 1)) * w.keys + warp * 16 + 2 * t;
  const bf16* p1 = w.weights + ((long long)b * nh + h0 + min(g + 8, gn - 1)) * w.keys + warp * 16 + 2 * t;
  float o[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
  auto scaled = [](uint32_t p, float f) {         // two weights times a power of two
    const __nv_bfloat162 v = __hmul2(*reinterpret_cast<const __nv_bfloat162*>(&p), __float2bfloat162_rn(f));
    return *reinterpret_cast<const uint32_t*>(&v);
  };
  const int d = x * 64 + g * 8;
  const bool there = d < vd;
  struct Rows {
    uint4 r[4];
    uint32_t p[4];
    float f0, f1;
  };
  auto fetch = [&](Rows& v, int c, int page) {
    const bf16* rows = (const bf16*)a.v_pages + (((long long)page * nkv + kv) * LLG_PAGE + warp * 16 + 2 * t) * vd + d;
#pragma unroll
    for (int r = 0; r < 4; ++r)
      v.r[r] = there ? *reinterpret_cast<const uint4*>(rows + (long long)((r & 1) + (r >> 1) * 8) * vd) : make_uint4(0, 0, 0, 0);
    v.p[0] = *reinterpret_cast<const uint32_t*>(p0 + c * CHUNK);
    v.p[1] = *reinterpret_cast<const uint32_t*>(p1 + c * CHUNK);
    v.p[2] = *reinterpret_cast<const uint32_t*>(p0 + c * CHUNK + 8);
    v.p[3] = *reinterpret_cast<const uint32_t*>(p1 + c * CHUNK + 8);
    v.f0 = ch[((long long)min(g, gn - 1) * all + c) * 2];
    v.f1 = ch[((long long)min(g + 8, gn - 1) * all + c) * 2];
  };
  auto add = [&](const Rows& v) {
    const float f0 = pow2_whole(v.f0 - m0), f1 = pow2_whole(v.f1 - m1);
    const uint32_t pa[4] = {scaled(v.p[0], f0), scaled(v.p[1], f1), scaled(v.p[2], f0), scaled(v.p[3], f1)};
    const uint32_t w0[4] = {v.r[0].x, v.r[0].y, v.r[0].z, v.r[0].w}, w1[4] = {v.r[1].x, v.r[1].y, v.r[1].z, v.r[1].w};
    const uint32_t w2[4] = {v.r[2].x, v.r[2].y, v.r[2].z, v.r[2].w}, w3[4] = {v.r[3].x, v.r[3].y, v.r[3].z, v.r[3].w};
#pragma unroll
    for (int j = 0; j < 8; ++j) {                 // element j of the four rows: the low or the high half of word j / 2
      const uint32_t sel = j & 1 ? 0x7632u : 0x5410u;
      mma_16816(o[j], pa, __byte_perm(w0[j / 2], w1[j / 2], sel), __byte_perm(w2[j / 2], w3[j / 2], sel));
    }
  };
  if (c0 < c1) {
    Rows va, vb;
    auto page_of = [&](int c) { return c < c1 ? page_at(a, slot, base + c * CHUNK) : 0; };
    int next = page_of(c0 + 1);
    fetch(va, c0, page_of(c0));
    for (int c = c0; c < c1; c += 2) {
      if (c + 1 < c1) fetch(vb, c + 1, next);
      next = page_of(c + 2);
      add(va);
      if (c + 1 >= c1) break;
      if (c + 2 < c1) fetch(va, c + 2, next);
      next = page_of(c + 3);
      add(vb);
    }
  }
  // column n of product j is element 64 x + 8 n + j; add the four warps up
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) merge[warp][g + (e >> 1) * 8][8 * (2 * t + (e & 1)) + j] = o[j][e];
  __syncthreads();
  const int dn = min(64, vd - x * 64);
  for (int idx = threadIdx.x; idx < gn * 64; idx += 128) {
    const int h = idx / 64, e = idx % 64;
    if (e < dn)
      a.part_o[(((long long)b * nh + h0 + h) * a.n_splits + split) * vd + x * 64 + e] =
          (merge[0][h][e] + merge[1][h][e]) + (merge[2][h][e] + merge[3][h][e]);
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

bool head_sizes_ok(int nh, int nkv, int hd, int vd) {
  return nh > 0 && nkv > 0 && nh % nkv == 0 && nh <= 128 && hd >= 16 && hd <= 128 && hd % 16 == 0 && vd >= 16 && vd <= 128 && vd % 16 == 0;
}

}  // namespace

// 1 when the kernels of this file take these sizes.
LLG_API int llg_attn_mix_prefill_mma_supported(int nh, int nkv, int hd, int vd) {
  MixCut p;
  return head_sizes_ok(nh, nkv, hd, vd) && plan_prefill(nh, nkv, hd, vd, &p);
}
LLG_API int llg_attn_mix_decode_mma_supported(int nh, int nkv, int hd, int vd) { return head_sizes_ok(nh, nkv, hd, vd); }

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

// scores [n_seqs][keys][nh] float32, weights [n_seqs][nh][keys] bfloat16 and chunks [n_seqs][nh][keys / 64][2] float32 are scratch;
// keys: a multiple of 64, no less than any sequence's keys (the new one included).
LLG_API int llg_attn_mix_decode_mma(const DecodeArgs* args, void* out, float* scores, void* weights, float* chunks, int keys,
                                    cudaStream_t stream) {
  const DecodeArgs& a = *args;
  const int vd = a.vd > 0 ? a.vd : a.hd;
  LLG_REQUIRE(head_sizes_ok(a.nh, a.nkv, a.hd, vd), "attn_mix_decode_mma: %d heads (%d) of %d and %d elements", a.nh, a.nkv, a.hd, vd);
  LLG_REQUIRE(a.scale > 0.f && a.softcap >= 0.f, "attn_mix_decode_mma: scale %g, cap %g", a.scale, a.softcap);
  LLG_REQUIRE(a.n_splits >= 1 && a.n_splits <= 65535 && a.n_seqs <= 65535, "attn_mix_decode_mma: grid too large");
  LLG_REQUIRE(a.window >= 0 && a.ring_pages > 0 && a.table_width >= a.ring_pages, "attn_mix_decode_mma: bad cache geometry");
  LLG_REQUIRE(keys > 0 && keys % CHUNK == 0 && scores && weights && chunks, "attn_mix_decode_mma: scratch for %d keys", keys);
  if (a.n_seqs <= 0) return 0;
  const MixScratch w{scores, (bf16*)weights, chunks, keys};
  const int rc = (a.nh / a.nkv + 15) / 16;
  // as many blocks as the GPU holds at once (four per multiprocessor), each with an equal share of its sequence's keys
  int shares = 4 * llg_sm_count() / (a.nkv * a.n_seqs);
  shares = shares < 1 ? 1 : shares > keys / CHUNK ? keys / CHUNK : shares;
  const dim3 sgrid(shares, a.nkv, a.n_seqs);
  if (a.hd <= 64) llg_launch(mix_scores_kernel<2>, sgrid, dim3(128), 0, stream, a, w);
  else llg_launch(mix_scores_kernel<4>, sgrid, dim3(128), 0, stream, a, w);
  const size_t smem = (size_t)(((a.nh + 3) & ~3) + CHUNK) * heads_stride(a.nh) * sizeof(float);
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(mix_weights_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return llg_fail("attn_mix_decode_mma: shared memory %zu: %s", smem, cudaGetErrorString(e));
  }
  llg_launch(mix_weights_kernel, dim3(keys / CHUNK, a.n_seqs), dim3(256), smem, stream, a, w);
  llg_launch(mix_values_kernel, dim3(a.n_splits, a.nkv * rc * ((vd + 63) / 64), a.n_seqs), dim3(128), 0, stream, a, w);
  attn_decode_reduce_kernel<bf16><<<dim3(a.nh, a.n_seqs), 64, 0, stream>>>(a.part_o, a.part_ml, (bf16*)out, a.nh, vd, a.n_splits, a.has_sink,
                                                                        a.sink_score, a.gate, a.sinks);
  return llg_check_launch("attn_mix_decode_mma");
}
