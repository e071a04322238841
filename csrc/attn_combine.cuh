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
  // every warp works out the factors of all splits (at most 32), one per lane
  const int lane = threadIdx.x & 31;
  const float2 mine = lane < splits ? *reinterpret_cast<const float2*>(ml + 2 * lane) : make_float2(-INFINITY, 0.f);
  const float gm = warp_max(mine.x);
  const float f = mine.x != -INFINITY ? __expf(mine.x - gm) : 0.f;
  float gl = warp_sum(mine.y * f);
  if (rule.sinks != nullptr) gl += __expf(rule.sinks[h] - gm);
  const float inv = gl > 0.f ? rule.out_scale / gl : 0.f;
  const float* o_row = part_o + static_cast<size_t>(bh) * splits * D;
  for (int d0 = threadIdx.x - lane; d0 < dv; d0 += blockDim.x) {
    const int d = d0 + lane;
    float o = 0.f;
#pragma unroll 8
    for (int s = 0; s < splits; ++s) {
      const float fs = __shfl_sync(0xffffffffu, f, s);
      if (fs != 0.f && d < dv) o = fmaf(o_row[static_cast<size_t>(s) * D + d], fs, o);
    }
    if (d < dv)
      out[static_cast<size_t>(b) * out_stride + static_cast<size_t>(h) * dv + d] =
          __float2bfloat16(o * inv * rule_gate<__nv_bfloat16>(rule, b, h, d));
  }
}

// The same for pairs of heads (AttnRule::pair): one CTA of 128 threads per (request, output head), dv <= 128.
static __global__ void __launch_bounds__(128)
attn_pair_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, __nv_bfloat16* __restrict__ out, int D, int dv,
                         int splits, int out_stride, int Hout, const AttnRule rule) {
  __shared__ float scratch[32];
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.x / Hout, h = blockIdx.x % Hout, lane = threadIdx.x & 31, d = threadIdx.x;
  float a[2];
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    const size_t bh = (static_cast<size_t>(b) * Hout + h) * 2 + m;
    const float* ml = part_ml + bh * splits * 2;
    const float2 mine = lane < splits ? *reinterpret_cast<const float2*>(ml + 2 * lane) : make_float2(-INFINITY, 0.f);
    const float gm = warp_max(mine.x);
    const float f = mine.x != -INFINITY ? __expf(mine.x - gm) : 0.f;
    const float gl = warp_sum(mine.y * f);
    const float* o_row = part_o + bh * splits * D;
    float o = 0.f;
#pragma unroll 8
    for (int s = 0; s < splits; ++s) {
      const float fs = __shfl_sync(0xffffffffu, f, s);
      if (fs != 0.f && d < dv) o = fmaf(o_row[static_cast<size_t>(s) * D + d], fs, o);
    }
    a[m] = gl > 0.f ? o / gl : 0.f;
  }
  const float x = d < dv ? fmaf(-rule.pair[0], a[1], a[0]) : 0.f;
  const float r = rule.pair_gain / sqrtf(block_sum<128>(x * x, scratch) / dv + rule.pair_eps);
  if (d < dv) out[static_cast<size_t>(b) * out_stride + static_cast<size_t>(h) * dv + d] = __float2bfloat16(x * r);
}

}  // namespace sb
