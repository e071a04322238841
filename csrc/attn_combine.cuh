// Second step of decode attention over several key ranges, shared by the decode kernels.
#pragma once

#include "attn_rule.cuh"

namespace sb {

inline AttnRule plain_rule() {
  AttnRule r = {};
  r.bytes = sizeof(AttnRule);
  r.window = 0x7fffffff;
  r.scale = r.out_scale = 1.f;
  return r;
}

// sigmoid of row t's gate for channel d of head h; 1 without a gate
template <typename T>
__device__ __forceinline__ float rule_gate(const AttnRule& r, long t, int h, int d) {
  if (r.gate == nullptr) return 1.f;
  const T* g = reinterpret_cast<const T*>(r.gate) + t * r.gate_pitch + static_cast<long>(h) * r.gate_width;
  return sigmoid_f(static_cast<float>(g[r.gate_width > 1 ? d : 0]));
}

// out[b, h, :] = sum_s o_s exp(m_s - M) / sum_s l_s exp(m_s - M) over the splits of one (request, head).
// dv: width of an output head (= D, or less where the kernel padded it). Sinks, output factor and gate as in AttnRule.
static __global__ void attn_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                           __nv_bfloat16* __restrict__ out, int D, int dv, int splits, int out_stride, int Hq,
                                           const AttnRule rule) {
  pdl_wait();
  pdl_launch_dependents();
  const int bh = blockIdx.x, b = bh / Hq, h = bh % Hq;
  const float* ml = part_ml + static_cast<size_t>(bh) * splits * 2;
  float gm = -INFINITY;
  for (int s = 0; s < splits; ++s) gm = fmaxf(gm, ml[2 * s]);
  float gl = 0.f;
  for (int s = 0; s < splits; ++s)
    if (ml[2 * s] != -INFINITY) gl += ml[2 * s + 1] * __expf(ml[2 * s] - gm);
  if (rule.sinks != nullptr) gl += __expf(rule.sinks[h] - gm);
  const float inv = gl > 0.f ? rule.out_scale / gl : 0.f;
  for (int d = threadIdx.x; d < dv; d += blockDim.x) {
    float o = 0.f;
    for (int s = 0; s < splits; ++s)
      if (ml[2 * s] != -INFINITY) o += part_o[(static_cast<size_t>(bh) * splits + s) * D + d] * __expf(ml[2 * s] - gm);
    out[static_cast<size_t>(b) * out_stride + static_cast<size_t>(h) * dv + d] =
        __float2bfloat16(o * inv * rule_gate<__nv_bfloat16>(rule, b, h, d));
  }
}

}  // namespace sb
