// Joins the partial results of a sequence's key splits (decode attention): the last kernel of the split forms that keep
// their partials in part_o / part_ml (DecodeArgs).  The sink joins the sum here, the gate multiplies the result.
#pragma once

namespace {

template <typename T>
__global__ void attn_decode_reduce_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                          T* __restrict__ out, int nh, int hd, int n_splits, int has_sink,
                                          float sink_score, const float* __restrict__ gate,
                                          const float* __restrict__ sinks) {
  // (hd: elements of a value head)
  const int h = blockIdx.x, b = blockIdx.y;
  if (sinks) sink_score = sinks[h];
  const long long base = ((long long)b * nh + h) * n_splits;
  float M = -INFINITY;
  for (int s = 0; s < n_splits; ++s) M = fmaxf(M, part_ml[(base + s) * 2]);
  if (has_sink) M = fmaxf(M, sink_score);
  float L = has_sink ? expf(sink_score - M) : 0.f;
  for (int s = 0; s < n_splits; ++s) {
    const float ms = part_ml[(base + s) * 2];
    if (ms != -INFINITY) L += expf(ms - M) * part_ml[(base + s) * 2 + 1];
  }
  float inv = L > 0.f ? 1.0f / L : 0.f;
  if (gate) inv *= gate[(long long)b * nh + h];
  for (int d = threadIdx.x; d < hd; d += blockDim.x) {
    float o = 0.f;
    for (int s = 0; s < n_splits; ++s) {
      const float ms = part_ml[(base + s) * 2];
      if (ms != -INFINITY) o += expf(ms - M) * part_o[(base + s) * hd + d];
    }
    out[((long long)b * nh + h) * hd + d] = from_f32<T>(o * inv);
  }
}

}  // namespace
