// Windowed attention over the paged cache on the CUDA cores: one warp per (query row, head), any head widths, bf16 or
// fp32 storage. It is the full-precision form of the tensor-core kernels (flash_window_sm100.cu for prompts,
// decode_attn_sm100.cu for single tokens) and takes the shapes they do not cover.
//
// Query row t belongs to request row_req[t] (null: request t) and stands at position row_pos[t]; attn_rule.cuh says what it
// sees and how its scores are made.
// Cache layout as everywhere: [num_slots, Hkv, D], slot = page * page_size + offset, pages from block_table[request]; v_pitch:
// elements between the value rows (a latent cache keeps one vector per token whose first DV elements are the value).
// Pairs of heads: a warp has one output head and computes its two attentions one after the other.
#include "attn_rule.cuh"

namespace sb {

constexpr int WA_WARPS = 4;
constexpr int WA_MAX_D = 1024;
constexpr int WA_ACC = WA_MAX_D / 32;

__device__ __forceinline__ float wa_load(const float* p) { return *p; }
__device__ __forceinline__ float wa_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void wa_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void wa_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

template <typename T, bool PAIR>
__global__ void __launch_bounds__(WA_WARPS * 32)
window_attn_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                   const int* __restrict__ block_table, const int* __restrict__ row_req, const int* __restrict__ row_pos,
                   T* __restrict__ out, int Hq, int Hkv, int D, int DV, int page_size, int max_pages, long q_stride, long out_stride,
                   long v_pitch, const AttnRule rule) {
  __shared__ float q_s[WA_WARPS][WA_MAX_D];
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long t = blockIdx.x;
  const int out_head = blockIdx.y * WA_WARPS + warp;
  if (out_head >= (PAIR ? Hq / 2 : Hq)) return;
  float first[PAIR ? WA_ACC : 1];  // the first attention of a pair
#pragma unroll
  for (int map = 0; map < (PAIR ? 2 : 1); ++map) {
  const int h = PAIR ? 2 * out_head + map : out_head;
  const int kvh = h / (Hq / Hkv);
  const int pos = row_pos[t];
  const int* bt = block_table + static_cast<long>(row_req != nullptr ? row_req[t] : t) * max_pages;
  const float slope = rule.slopes != nullptr ? rule.slopes[h] : 0.f;
  __syncwarp();
  for (int d = lane; d < D; d += 32) q_s[warp][d] = wa_load(q + t * q_stride + static_cast<long>(h) * D + d);
  __syncwarp();

  float m = -INFINITY, l = 0.f, acc[WA_ACC];
#pragma unroll
  for (int i = 0; i < WA_ACC; ++i) acc[i] = 0.f;
  const int lo = rule_first_key(rule, pos);  // first key of the window
  const int kept = min(rule.keep_first, lo);  // kept keys in front of it
  const int nkeys = kept + (pos - lo + 1);
  for (int n0 = 0; n0 < nkeys; n0 += 32) {
    const int n = n0 + lane;
    const int key = n < kept ? n : lo + n - kept;
    long slot = 0;
    float s = -INFINITY;
    if (n < nkeys) {
      slot = static_cast<long>(bt[key / page_size]) * page_size + key % page_size;
      const T* kr = k_cache + (slot * Hkv + kvh) * D;
      float dot = 0.f;
      for (int d = 0; d < D; ++d) dot = fmaf(q_s[warp][d], wa_load(kr + d), dot);
      s = dot * rule.scale;
      if (rule.softcap > 0.f) s = rule.softcap * tanhf(s / rule.softcap);
      if (rule.bias != nullptr) s += rule.bias[static_cast<long>(min(pos - key, rule.bias_rows - 1)) * Hq + h];
      s -= slope * static_cast<float>(pos - key);
    }
    const float nm = fmaxf(m, warp_max(s));
    const float p = n < nkeys ? expf(s - nm) : 0.f;
    const float corr = m == -INFINITY ? 0.f : expf(m - nm);
    l = l * corr + warp_sum(p);
    m = nm;
#pragma unroll
    for (int i = 0; i < WA_ACC; ++i) acc[i] *= corr;
    const int cnt = min(32, nkeys - n0);
    for (int j = 0; j < cnt; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const long sj = __shfl_sync(0xffffffffu, slot, j);
      const T* vr = v_cache + (sj * Hkv + kvh) * v_pitch;
#pragma unroll
      for (int i = 0; i < WA_ACC; ++i)
        if (lane + 32 * i < DV) acc[i] = fmaf(pj, wa_load(vr + lane + 32 * i), acc[i]);
    }
  }
  if constexpr (PAIR) {
    const float norm = 1.f / l;
    if (map == 0) {
#pragma unroll
      for (int i = 0; i < WA_ACC; ++i) first[i] = acc[i] * norm;
      continue;
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < WA_ACC; ++i) {
      first[i] = lane + 32 * i < DV ? fmaf(-rule.pair[0], acc[i] * norm, first[i]) : 0.f;
      ss = fmaf(first[i], first[i], ss);
    }
    const float r = rule.pair_gain / sqrtf(warp_sum(ss) / DV + rule.pair_eps);
#pragma unroll
    for (int i = 0; i < WA_ACC; ++i)
      if (lane + 32 * i < DV) wa_store(out + t * out_stride + static_cast<long>(out_head) * DV + lane + 32 * i, first[i] * r);
    return;
  }
  if (rule.sinks != nullptr) l += expf(rule.sinks[h] - m);
  const float inv = rule.out_scale / l;  // a row always sees its own key: l > 0
  const T* gate = reinterpret_cast<const T*>(rule.gate) + (rule.gate != nullptr ? t * rule.gate_pitch + static_cast<long>(h) * rule.gate_width : 0);
#pragma unroll
  for (int i = 0; i < WA_ACC; ++i) {
    const int d = lane + 32 * i;
    if (d >= DV) continue;
    const float g = rule.gate != nullptr ? sigmoid_f(wa_load(gate + (rule.gate_width > 1 ? d : 0))) : 1.f;
    wa_store(out + t * out_stride + static_cast<long>(h) * DV + d, acc[i] * inv * g);
  }
  }
}

}  // namespace sb

extern "C" int sb_window_attn(const void* q, const void* k_cache, const void* v_cache, const int* block_table, const int* row_req,
                              const int* row_pos, void* out, int T, int Hq, int Hkv, int D, int DV, int page_size, int max_pages,
                              long q_stride, long out_stride, long v_pitch, const void* rule, int f32, cudaStream_t s) {
  if (T == 0) return 0;
  const sb::AttnRule* r = (const sb::AttnRule*)rule;
  if (Hkv <= 0 || Hq % Hkv != 0 || D <= 0 || DV <= 0 || D > sb::WA_MAX_D || DV > sb::WA_MAX_D || !rule_ok(r) || !rule_pairs_ok(r, Hq / Hkv))
    return (int)cudaErrorInvalidValue;
  const int heads = r->pair != nullptr ? Hq / 2 : Hq;
  const dim3 grid(T, (heads + sb::WA_WARPS - 1) / sb::WA_WARPS);
  using bf16 = __nv_bfloat16;
  const bool pair = r->pair != nullptr;
  if (f32)
    return (int)sb::launch_pdl(pair ? sb::window_attn_kernel<float, true> : sb::window_attn_kernel<float, false>, grid, dim3(sb::WA_WARPS * 32), 0, s, (const float*)q, (const float*)k_cache,
                               (const float*)v_cache, block_table, row_req, row_pos, (float*)out, Hq, Hkv, D, DV, page_size, max_pages,
                               q_stride, out_stride, v_pitch, *r);
  return (int)sb::launch_pdl(pair ? sb::window_attn_kernel<bf16, true> : sb::window_attn_kernel<bf16, false>, grid, dim3(sb::WA_WARPS * 32), 0, s, (const bf16*)q, (const bf16*)k_cache,
                             (const bf16*)v_cache, block_table, row_req, row_pos, (bf16*)out, Hq, Hkv, D, DV, page_size, max_pages, q_stride,
                             out_stride, v_pitch, *r);
}
