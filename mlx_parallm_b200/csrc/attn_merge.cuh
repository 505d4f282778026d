// Merge of a decode step's partial attention sums (keys split over CTAs), shared by the attention kernels that split keys.
#pragma once
#include "common.cuh"

namespace b200p {

constexpr float LOG2E = 1.4426950408889634f;

// out[e's token, h, :] = out_scale * (sum_s o_s 2^(m_s - m)) / (2^(sink log2e - m) + sum_s l_s 2^(m_s - m)), m the largest of them;
// part_o [e, h, splits, dv], part_ms [e, h, splits, 2] = (running max in base-2 units, sum), (-inf, 0) for a share without keys.
// cu NULL: entry e is token e.
template <typename T>
__global__ void attn_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ms,
                                  const int32_t* __restrict__ cu, const float* __restrict__ sink, T* __restrict__ out,
                                  int64_t ld_out, float out_scale, int H, int dv, int splits, const float* __restrict__ gate,
                                  int64_t ldg) {
  const int e = blockIdx.x, h = blockIdx.y;
  if (cu && cu[e + 1] - cu[e] <= 0) return;
  const int64_t t = cu ? cu[e] : e;
  const int64_t base = ((int64_t)e * H + h) * splits;
  float m = sink ? sink[h] * LOG2E : -INFINITY;
  for (int sidx = 0; sidx < splits; ++sidx) m = fmaxf(m, part_ms[(base + sidx) * 2]);
  float den = sink ? exp2f(sink[h] * LOG2E - m) : 0.f;
  for (int sidx = 0; sidx < splits; ++sidx) {
    const float ms = part_ms[(base + sidx) * 2];
    if (ms != -INFINITY) den += part_ms[(base + sidx) * 2 + 1] * exp2f(ms - m);
  }
  const float inv = out_scale / den;
  for (int c = threadIdx.x; c < dv; c += blockDim.x) {
    float a = 0.f;
    for (int sidx = 0; sidx < splits; ++sidx) {
      const float ms = part_ms[(base + sidx) * 2];
      if (ms != -INFINITY) a = fmaf(part_o[(base + sidx) * dv + c], exp2f(ms - m), a);
    }
    const float gz = gate ? 1.f / (1.f + expf(-gate[t * ldg + (int64_t)h * dv + c])) : 1.f;
    out[t * ld_out + (int64_t)h * dv + c] = Tr<T>::from_f(a * inv * gz);
  }
}

}  // namespace b200p
