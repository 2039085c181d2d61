// Attention whose scores are capped and mixed over the heads ahead of the softmax:
//
//   s_h = cap tanh(scale q_h . k / cap)   (cap > 0),    s'_h = sum_g mix[h][g] s_g   (mix given),
//   p_h = softmax of s'_h over the visible keys, a sink (where there is one) in the denominator
//
// Every head's weights depend on all heads' scores, so a block works on all query heads of its queries at once.  The
// contract is that of the other attention kernels (kernel_args.h: PrefillArgs, DecodeArgs): value heads of another size,
// sinks, gates, windows and chunks by argument.
//
// The kernels of this part run on the CUDA cores in float32 arithmetic, for float32 and bfloat16 storage and any head
// size up to 384: the true 32-bit path, and what sizes take that the tensor-core kernels do not.
//
//   attn_mix_prefill_simt : BQ queries of all heads per block; key tiles of 32.
//   attn_mix_decode_simt  : one new token per sequence; the keys of a sequence are split over blocks whose partial
//                           results attn_decode_reduce joins.
#include "common.cuh"
#include "kernel_args.h"
#include "attention_reduce.cuh"

LLG_API const char* llg_last_error() { return g_llg_error; }

namespace {

constexpr int MK = 32;            // keys per tile (one per lane)
constexpr int MIX_THREADS = 256;
constexpr int MIX_MAX_HEAD = 384;

// What the walk over a sequence's keys needs; keys at positions from `lb` on lie in the step's packed buffers, earlier
// ones in the cache pages.
struct MixWalk {
  const void* q;                  // the tile's first query: [.][nh][hd]
  const void *k_new, *v_new;      // null: every key is in the pages
  const void *k_pages, *v_pages;
  const int* page_table;
  int table_width, ring_pages, slot;
  int tok0, lb;                   // row of k_new that holds position lb
  int nq, pos0, k_begin, k_end;   // queries, position of the first, keys [k_begin, k_end)
  int nh, nkv, hd, vd;
  float scale, softcap;
  const float* mix;
  int window, chunked;
};

// shared memory: Q [nh][BQ][hd], acc [nh][BQ][vd], S and P [nh][BQ][MK], m, l, corr [nh][BQ], KV [MK][max(hd, vd) + 1]
template <int BQ>
__host__ __device__ inline size_t mix_floats(int nh, int hd, int vd) {
  return (size_t)nh * BQ * (hd + vd + 2 * MK + 3) + (size_t)MK * ((hd > vd ? hd : vd) + 1);
}

template <typename T, int BQ>
__device__ __forceinline__ void mix_walk(const MixWalk& w, float* sm, float*& acc, float*& m, float*& l) {
  __shared__ long long src_off[MK];
  __shared__ int src_new[MK];
  const int nh = w.nh, hd = w.hd, vd = w.vd, G = nh / w.nkv;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  constexpr int WARPS = MIX_THREADS / 32;
  float* Q = sm;
  acc = Q + nh * BQ * hd;
  float* S = acc + nh * BQ * vd;
  float* P = S + nh * BQ * MK;
  m = P + nh * BQ * MK;
  l = m + nh * BQ;
  float* corr = l + nh * BQ;
  float* KV = corr + nh * BQ;
  const T* q = (const T*)w.q;
  for (int idx = tid; idx < nh * BQ * hd; idx += MIX_THREADS) {
    const int d = idx % hd, r = idx / hd, qi = r % BQ, h = r / BQ;
    Q[idx] = qi < w.nq ? to_f32(q[((long long)qi * nh + h) * hd + d]) : 0.f;
  }
  for (int idx = tid; idx < nh * BQ * vd; idx += MIX_THREADS) acc[idx] = 0.f;
  for (int idx = tid; idx < nh * BQ; idx += MIX_THREADS) {
    m[idx] = -INFINITY;
    l[idx] = 0.f;
  }
  const int k0 = w.k_begin / MK * MK;
  for (int kt = k0; kt < w.k_end; kt += MK) {
    for (int g = 0; g < w.nkv; ++g) {
      __syncthreads();
      if (tid < MK) {
        const int kp = kt + tid;
        int sn = -1;
        long long off = 0;
        if (kp < w.k_end) {
          if (w.k_new && kp >= w.lb) {
            sn = 1;
            off = (long long)(w.tok0 + kp - w.lb) * w.nkv + g;
          } else {
            sn = 0;
            off = kv_row(w.page_table, w.table_width, w.ring_pages, w.slot, kp, g, w.nkv);
          }
        }
        src_new[tid] = sn;
        src_off[tid] = off;
      }
      __syncthreads();
      for (int idx = tid; idx < MK * hd; idx += MIX_THREADS) {
        const int j = idx / hd, d = idx - j * hd;
        const int sn = src_new[j];
        KV[j * (hd + 1) + d] = sn < 0 ? 0.f : to_f32(((const T*)(sn ? w.k_new : w.k_pages))[src_off[j] * hd + d]);
      }
      __syncthreads();
      for (int r = warp; r < G * BQ; r += WARPS) {
        const float* qr = Q + (g * G * BQ + r) * hd;
        const float* kr = KV + lane * (hd + 1);
        float s = 0.f;
        for (int d = 0; d < hd; ++d) s = fmaf(qr[d], kr[d], s);
        s *= w.scale;
        if (w.softcap > 0.f) s = w.softcap * tanhf(s / w.softcap);
        S[(g * G * BQ + r) * MK + lane] = s;
      }
    }
    __syncthreads();
    // mix, mask, running maximum and weights: a warp per (head, query), a lane per key
    const int kp = kt + lane;
    for (int r = warp; r < nh * BQ; r += WARPS) {
      const int h = r / BQ, qi = r % BQ, qpos = w.pos0 + qi;
      float s;
      if (w.mix) {
        s = 0.f;
        for (int g = 0; g < nh; ++g) s = fmaf(w.mix[h * nh + g], S[(g * BQ + qi) * MK + lane], s);
      } else {
        s = S[r * MK + lane];
      }
      const bool valid = qi < w.nq && kp < w.k_end && kp <= qpos && kp >= mask_first(qpos, w.window, w.chunked);
      if (!valid) s = -INFINITY;
      const float mo = m[r], mn = fmaxf(mo, warp_max(s));
      const float p = valid ? expf(s - mn) : 0.f;
      const float c = mn == -INFINITY ? 1.f : expf(mo - mn);
      const float sum = warp_sum(p);
      P[r * MK + lane] = p;
      __syncwarp();
      if (lane == 0) {
        m[r] = mn;
        l[r] = l[r] * c + sum;
        corr[r] = c;
      }
    }
    for (int g = 0; g < w.nkv; ++g) {
      __syncthreads();
      if (tid < MK && src_new[tid] == 0) src_off[tid] = kv_row(w.page_table, w.table_width, w.ring_pages, w.slot, kt + tid, g, w.nkv);
      if (tid < MK && src_new[tid] == 1) src_off[tid] = (long long)(w.tok0 + kt + tid - w.lb) * w.nkv + g;
      __syncthreads();
      for (int idx = tid; idx < MK * vd; idx += MIX_THREADS) {
        const int j = idx / vd;
        const int sn = src_new[j];
        KV[idx] = sn < 0 ? 0.f : to_f32(((const T*)(sn ? w.v_new : w.v_pages))[src_off[j] * vd + idx - j * vd]);
      }
      __syncthreads();
      for (int idx = tid; idx < G * BQ * vd; idx += MIX_THREADS) {
        const int d = idx % vd, r = g * G * BQ + idx / vd;
        const float* pr = P + r * MK;
        float o = acc[r * vd + d] * corr[r];
#pragma unroll 8
        for (int j = 0; j < MK; ++j) o = fmaf(pr[j], KV[j * vd + d], o);
        acc[r * vd + d] = o;
      }
    }
  }
  __syncthreads();
}

template <typename T, int BQ>
__global__ void __launch_bounds__(MIX_THREADS) attn_mix_prefill_simt_kernel(PrefillArgs a) {
  extern __shared__ float sm[];
  const int b = a.tiles[2 * blockIdx.x], q_off = a.tiles[2 * blockIdx.x + 1] + (int)blockIdx.y * BQ;
  const int tok0 = a.cu_tokens[b], t_b = a.cu_tokens[b + 1] - tok0;
  if (q_off >= t_b) return;
  const int vd = a.vd > 0 ? a.vd : a.hd;
  MixWalk w;
  w.nq = min(BQ, t_b - q_off);
  w.lb = a.len_before[b];
  w.slot = a.slots[b];
  w.tok0 = tok0;
  w.pos0 = w.lb + q_off;
  w.k_end = w.pos0 + w.nq;
  w.k_begin = mask_first(w.pos0, a.window, a.chunked);
  w.q = (const T*)a.q + (long long)(tok0 + q_off) * a.nh * a.hd;
  w.k_new = a.k_new; w.v_new = a.v_new; w.k_pages = a.k_pages; w.v_pages = a.v_pages;
  w.page_table = a.page_table; w.table_width = a.table_width; w.ring_pages = a.ring_pages;
  w.nh = a.nh; w.nkv = a.nkv; w.hd = a.hd; w.vd = vd;
  w.scale = a.scale; w.softcap = a.softcap; w.mix = a.head_mix; w.window = a.window; w.chunked = a.chunked;
  float *acc, *m, *l;
  mix_walk<T, BQ>(w, sm, acc, m, l);
  T* out = (T*)a.out + (long long)(tok0 + q_off) * a.nh * vd;
  for (int idx = threadIdx.x; idx < a.nh * BQ * vd; idx += MIX_THREADS) {
    const int d = idx % vd, r = idx / vd, qi = r % BQ, h = r / BQ;
    if (qi >= w.nq) continue;
    float li = l[r], keep = 1.f;
    if (a.has_sink) {
      const float sink = a.sinks ? a.sinks[h] : a.sink_score;
      const float m_all = fmaxf(m[r], sink);
      keep = expf(m[r] - m_all);
      li = li * keep + expf(sink - m_all);
    }
    float inv = li > 0.f ? keep / li : 0.f;
    if (a.gate) inv *= a.gate[(long long)(tok0 + q_off + qi) * a.nh + h];
    out[((long long)qi * a.nh + h) * vd + d] = from_f32<T>(acc[idx] * inv);
  }
}

template <typename T>
__global__ void __launch_bounds__(MIX_THREADS) attn_mix_decode_simt_kernel(DecodeArgs a) {
  extern __shared__ float sm[];
  const int split = blockIdx.x, b = blockIdx.y;
  const int vd = a.vd > 0 ? a.vd : a.hd;
  const int len = a.len_before[b] + 1;
  const int lo = mask_first(len - 1, a.window, a.chunked);
  const int t0 = lo / MK, t_end = (len + MK - 1) / MK;
  const int per = (t_end - t0 + a.n_splits - 1) / a.n_splits;
  const int my0 = min(t_end, t0 + split * per), my1 = min(t_end, my0 + per);
  MixWalk w;
  w.nq = 1;
  w.lb = 0;
  w.tok0 = 0;
  w.slot = a.slots[b];
  w.pos0 = len - 1;
  w.k_begin = my0 * MK;
  w.k_end = min(len, my1 * MK);
  w.q = (const T*)a.q + (long long)b * a.nh * a.hd;
  w.k_new = nullptr; w.v_new = nullptr; w.k_pages = a.k_pages; w.v_pages = a.v_pages;
  w.page_table = a.page_table; w.table_width = a.table_width; w.ring_pages = a.ring_pages;
  w.nh = a.nh; w.nkv = a.nkv; w.hd = a.hd; w.vd = vd;
  w.scale = a.scale; w.softcap = a.softcap; w.mix = a.head_mix; w.window = a.window; w.chunked = a.chunked;
  float *acc, *m, *l;
  mix_walk<T, 1>(w, sm, acc, m, l);
  for (int idx = threadIdx.x; idx < a.nh * vd; idx += MIX_THREADS) {
    const int h = idx / vd, d = idx - h * vd;
    a.part_o[(((long long)b * a.nh + h) * a.n_splits + split) * vd + d] = acc[idx];
  }
  for (int h = threadIdx.x; h < a.nh; h += MIX_THREADS) {
    const long long p = ((long long)b * a.nh + h) * a.n_splits + split;
    a.part_ml[p * 2] = m[h];
    a.part_ml[p * 2 + 1] = l[h];
  }
}

constexpr size_t MIX_SMEM_MAX = 220 * 1024;

template <typename K>
int mix_attr(K kernel, size_t smem, const char* what) {
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return llg_fail("%s: shared memory %zu: %s", what, smem, cudaGetErrorString(e));
  return 0;
}

int check_mix(const char* what, int nh, int nkv, int hd, int vd, float scale, float softcap, int window, int ring, int width) {
  LLG_REQUIRE(nh > 0 && nkv > 0 && nh % nkv == 0, "%s: %d heads are no multiple of %d key/value heads", what, nh, nkv);
  LLG_REQUIRE(hd > 0 && hd <= MIX_MAX_HEAD && vd > 0 && vd <= MIX_MAX_HEAD, "%s: head sizes %d and %d are outside [1, %d]", what, hd, vd, MIX_MAX_HEAD);
  LLG_REQUIRE(scale > 0.f && softcap >= 0.f, "%s: scale %g, cap %g", what, scale, softcap);
  LLG_REQUIRE(window >= 0 && ring > 0 && width >= ring, "%s: bad cache geometry", what);
  return 0;
}

}  // namespace

// 1 when these kernels take the sizes: a block keeps one query of all heads in shared memory.
LLG_API int llg_attn_mix_simt_supported(int nh, int hd, int vd) {
  return nh > 0 && hd > 0 && hd <= MIX_MAX_HEAD && vd > 0 && vd <= MIX_MAX_HEAD && mix_floats<1>(nh, hd, vd) * sizeof(float) <= MIX_SMEM_MAX;
}

// tile_queries: queries per entry of `tiles`; a block takes 1, 2, 4 or 8 of them, what shared memory holds.
LLG_API int llg_attn_mix_prefill_simt(const PrefillArgs* args, int tile_queries, int dtype, cudaStream_t stream) {
  const PrefillArgs& a = *args;
  const int vd = a.vd > 0 ? a.vd : a.hd;
  if (check_mix("attn_mix_prefill", a.nh, a.nkv, a.hd, vd, a.scale, a.softcap, a.window, a.ring_pages, a.table_width)) return 1;
  LLG_REQUIRE(tile_queries > 0 && tile_queries % 8 == 0, "attn_mix_prefill: tiles of %d queries", tile_queries);
  LLG_REQUIRE(llg_attn_mix_simt_supported(a.nh, a.hd, vd), "attn_mix_prefill: %d heads of %d and %d elements do not fit shared memory", a.nh, a.hd, vd);
  LLG_REQUIRE(dtype == LLG_F32 || dtype == LLG_BF16, "attn_mix_prefill: unknown dtype %d", dtype);
  if (a.n_tiles <= 0) return 0;
#define GO(T, B)                                                                                              \
  do {                                                                                                        \
    const size_t smem = mix_floats<B>(a.nh, a.hd, vd) * sizeof(float);                                        \
    if (smem <= MIX_SMEM_MAX) {                                                                               \
      if (mix_attr(attn_mix_prefill_simt_kernel<T, B>, smem, "attn_mix_prefill")) return 1;                   \
      attn_mix_prefill_simt_kernel<T, B><<<dim3(a.n_tiles, tile_queries / B), MIX_THREADS, smem, stream>>>(a); \
      return llg_check_launch("attn_mix_prefill_simt");                                                       \
    }                                                                                                         \
  } while (0)
  if (dtype == LLG_F32) { GO(float, 8); GO(float, 4); GO(float, 2); GO(float, 1); }
  else { GO(__nv_bfloat16, 8); GO(__nv_bfloat16, 4); GO(__nv_bfloat16, 2); GO(__nv_bfloat16, 1); }
#undef GO
  return llg_fail("attn_mix_prefill: no block size fits");
}

LLG_API int llg_attn_mix_decode_simt(const DecodeArgs* args, void* out, int dtype, cudaStream_t stream) {
  const DecodeArgs& a = *args;
  const int vd = a.vd > 0 ? a.vd : a.hd;
  if (check_mix("attn_mix_decode", a.nh, a.nkv, a.hd, vd, a.scale, a.softcap, a.window, a.ring_pages, a.table_width)) return 1;
  LLG_REQUIRE(a.n_splits >= 1 && a.n_splits <= 65535 && a.n_seqs <= 65535, "attn_mix_decode: grid too large");
  LLG_REQUIRE(llg_attn_mix_simt_supported(a.nh, a.hd, vd), "attn_mix_decode: %d heads of %d and %d elements do not fit shared memory", a.nh, a.hd, vd);
  if (a.n_seqs <= 0) return 0;
  const size_t smem = mix_floats<1>(a.nh, a.hd, vd) * sizeof(float);
#define GO(T)                                                                                                          \
  do {                                                                                                                 \
    if (mix_attr(attn_mix_decode_simt_kernel<T>, smem, "attn_mix_decode")) return 1;                                   \
    attn_mix_decode_simt_kernel<T><<<dim3(a.n_splits, a.n_seqs), MIX_THREADS, smem, stream>>>(a);                      \
    attn_decode_reduce_kernel<T><<<dim3(a.nh, a.n_seqs), 64, 0, stream>>>(a.part_o, a.part_ml, (T*)out, a.nh, vd, a.n_splits, \
                                                                         a.has_sink, a.sink_score, a.gate, a.sinks);   \
  } while (0)
  if (dtype == LLG_F32) GO(float);
  else if (dtype == LLG_BF16) GO(__nv_bfloat16);
  else return llg_fail("attn_mix_decode: unknown dtype %d", dtype);
#undef GO
  return llg_check_launch("attn_mix_decode_simt");
}
