// What the attention kernels over the paged cache have in common: which keys a query sees, how its scores are made, what
// happens to its output. Filled on the host (slime_b200/ops/window_attention.py::Rule has the same layout).
//
//   query at position i sees key j  iff  j <= i  and  (j >= max(i - window + 1, chunk * floor(i / chunk))  or  j < keep_first)
//   s = scale * q.k;   s = softcap * tanh(s / softcap);   s += bias[i - j][head];   s -= slopes[head] * (i - j)
//   output = out_scale * sigmoid(gate) * softmax(s, sinks[head]) v
//
// Pairs (differential attention): query heads 2 i and 2 i + 1 are two attentions a1, a2 over the same values, and output head i is
//   d / rms(d) * pair_gain  with  d = a1 - pair[0] * a2  and  rms(d) = sqrt(mean(d^2) + pair_eps)
#pragma once

#include "common.cuh"

namespace sb {

struct AttnRule {
  int bytes;              // sizeof(AttnRule) as the caller sees it
  int window, keep_first;
  int chunk;              // 0: no chunks
  float scale, out_scale;
  float softcap;          // 0: scores are not capped
  int bias_rows;          // distances from bias_rows - 1 on share the last row
  int gate_width;         // gate columns of a head: 1, or the value width
  float pair_gain;
  long gate_pitch;        // elements between rows of gate
  float pair_eps;
  int reserved;
  const float* slopes;    // [Hq] or null
  const float* sinks;     // [Hq] score of an extra softmax column that has no value, or null
  const float* bias;      // [bias_rows, Hq] or null
  const void* gate;       // logits, rows as q and type of q, column head * gate_width (+ channel), or null
  const float* pair;      // one number, or null: every query head has an output of its own
};

__device__ __forceinline__ int rule_first_key(const AttnRule& r, int pos) {
  const int w = r.window > pos ? 0 : pos - r.window + 1;
  return r.chunk > 0 ? max(w, pos / r.chunk * r.chunk) : w;
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

// c * tanh(x * scale / c) in units of log2 e from the raw product x: c2 - 2 c2 / (1 + 2^(k x)) with c2 = c log2 e and
// k = 2 scale log2 e / c. 2^60 stands for anything larger: 1 / 2^60 vanishes beside 1 in fp32.
__device__ __forceinline__ float cap_exp2(float x, float k) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(fminf(x * k, 60.f)));
  return r + 1.f;
}
__device__ __forceinline__ float fast_rcp(float x) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

}  // namespace sb

static inline bool rule_ok(const sb::AttnRule* r) {
  return r != nullptr && r->bytes == static_cast<int>(sizeof(sb::AttnRule)) && r->window >= 1 && r->keep_first >= 0 && r->chunk >= 0 &&
         r->softcap >= 0.f && r->scale > 0.f && (r->bias == nullptr || r->bias_rows >= 1) && (r->gate == nullptr || r->gate_width >= 1) &&
         (r->pair == nullptr || (r->gate == nullptr && r->sinks == nullptr && r->bias == nullptr && r->slopes == nullptr && r->softcap == 0.f));
}

// Pairs need the two heads of each to share their keys' head.
static inline bool rule_pairs_ok(const sb::AttnRule* r, int group) { return r->pair == nullptr || group % 2 == 0; }
