// Gated delta rule over per-request recurrent states. Per head, with S [D, DV] in fp32:
//
//     S <- g S        u = beta (v - S^T k)        S <- S + k u^T        o = S^T q
//
// q, k, v are projections that passed a short causal convolution over time (per channel) and silu; q and k are unit vectors
// (q also times D^-1/2); head h uses q / k head h / (H / G). The decay g = exp(-exp(A_log) softplus(a + dt_bias)) is one number
// per head or one per key channel; beta = sigmoid(b). Everything is fp32 behind the projections.
//
//   sb_delta_prep    packed rows -> fp32 q, k, v, decay, beta and q.k of every token
//   sb_delta_scan    the recurrence over the rows of every request, states read and left in their slots
//   sb_head_gate     RMS norm of every head's output, its gate, bf16 / fp32 result
//   sb_delta_step    all of the above for one token per request, one launch
//
// The recurrence is evaluated token by token in registers, so a result does not depend on where a prompt was cut. Inputs that
// the convolution still needs live in a ring of `taps` rows per slot (row = position mod taps): the current token's row is never
// one that a reader of the same launch needs.
#include "common.cuh"

namespace sb {

constexpr int DR_MAX = 256;       // widest query / key or value head
constexpr int DR_MAX_TAPS = 16;

__device__ __forceinline__ float dr_load(const float* p) { return *p; }
__device__ __forceinline__ float dr_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void dr_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void dr_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float dr_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float dr_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float dr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float dr_decay(float rate, float z) { return expf(-rate * dr_softplus(z)); }

// Inputs of one layer, element type T (bf16 or fp32); rows of the projections are `pitch` elements apart.
struct DeltaIn {
  const void *q, *k, *v, *a, *b;  // [T, G D], [T, G D], [T, H DV], [T, H or H D], [T, H]
  long pitch, a_pitch, b_pitch;
  const void* conv;               // [2 G D + H DV, taps], channels in the order q, k, v
  const float *A_log, *dt_bias;   // [H], [H or H D]
  void* ring;                     // [slots, taps, 2 G D + H DV]
  float* state;                   // [slots, H, D, DV]
  int H, G, D, DV, taps, per_channel;
};

// Input of convolution channel c (column `col` of the projection x) at position `at`: from the pass's rows when it has
// the token, from the ring when an earlier pass had it, zero in front of the sequence. row0: row of position p0.
template <typename T>
__device__ __forceinline__ float dr_tap(const T* x, long pitch, int col, const T* ring, int C, int taps, int c, int at, int p0, long row0) {
  if (at >= p0) return dr_load(x + (row0 + at - p0) * pitch + col);
  return at >= 0 ? dr_load(ring + static_cast<long>(at % taps) * C + c) : 0.f;
}

// One warp per (run of tokens, vector): first the G query / key pairs, then the H values, then the H decays.
template <typename T>
__global__ void __launch_bounds__(128)
delta_prep_kernel(const __grid_constant__ DeltaIn a, const int4* __restrict__ runs, const int4* __restrict__ segs,
                  float* __restrict__ q_out, float* __restrict__ k_out, float* __restrict__ v_out, float* __restrict__ g_out,
                  float* __restrict__ beta_out, float* __restrict__ qk_out) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, vec = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (vec >= a.G + 2 * a.H) return;
  const int4 run = runs[blockIdx.x];  // first row, tokens, first position, request
  const int4 seg = segs[run.w];       // first row, tokens, first position, state slot
  const int H = a.H, G = a.G, D = a.D, DV = a.DV, taps = a.taps, C = 2 * G * D + H * DV;
  const T* ring = reinterpret_cast<const T*>(a.ring) + static_cast<long>(seg.w) * taps * C;
  const T* conv = reinterpret_cast<const T*>(a.conv);
  auto conv_at = [&](const T* x, int col, int c, int pos) {
    float y = 0.f;
    for (int s = 0; s < taps; ++s)
      y = fmaf(dr_load(conv + static_cast<long>(c) * taps + taps - 1 - s), dr_tap(x, a.pitch, col, ring, C, taps, c, pos - s, seg.z, seg.x), y);
    return dr_silu(y);
  };
  for (int i = 0; i < run.y; ++i) {
    const long row = run.x + i;
    const int pos = run.z + i;
    if (vec < G) {
      float q[DR_MAX / 32], k[DR_MAX / 32], qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
      for (int j = 0; j < DR_MAX / 32; ++j) {
        const int d = lane + 32 * j;
        q[j] = k[j] = 0.f;
        if (d < D) {
          q[j] = conv_at(reinterpret_cast<const T*>(a.q), vec * D + d, vec * D + d, pos);
          k[j] = conv_at(reinterpret_cast<const T*>(a.k), vec * D + d, (G + vec) * D + d, pos);
          qq = fmaf(q[j], q[j], qq);
          kk = fmaf(k[j], k[j], kk);
          qk = fmaf(q[j], k[j], qk);
        }
      }
      const float rq = 1.f / sqrtf(warp_sum(qq) + 1e-6f) / sqrtf(static_cast<float>(D)), rk = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
      qk = warp_sum(qk) * rq * rk;
#pragma unroll
      for (int j = 0; j < DR_MAX / 32; ++j) {
        const int d = lane + 32 * j;
        if (d < D) {
          q_out[(row * G + vec) * D + d] = q[j] * rq;
          k_out[(row * G + vec) * D + d] = k[j] * rk;
        }
      }
      if (lane == 0) qk_out[row * G + vec] = qk;
    } else if (vec < G + H) {
      const int h = vec - G;
      for (int d = lane; d < DV; d += 32)
        v_out[(row * H + h) * DV + d] = conv_at(reinterpret_cast<const T*>(a.v), h * DV + d, 2 * G * D + h * DV + d, pos);
      if (lane == 0) beta_out[row * H + h] = dr_sigmoid(dr_load(reinterpret_cast<const T*>(a.b) + row * a.b_pitch + h));
    } else {
      const int h = vec - G - H;
      const float rate = expf(a.A_log[h]);
      const T* ap = reinterpret_cast<const T*>(a.a) + row * a.a_pitch;
      if (a.per_channel) {
        for (int d = lane; d < D; d += 32)
          g_out[(row * H + h) * D + d] = dr_decay(rate, dr_load(ap + h * D + d) + a.dt_bias[h * D + d]);
      } else if (lane == 0) {
        g_out[row * H + h] = dr_decay(rate, dr_load(ap + h) + a.dt_bias[h]);
      }
    }
  }
}

// V adjacent elements as floats, and back.
template <int V>
__device__ __forceinline__ void dr_load_v(const float* p, float (&f)[V]) {
  if constexpr (V == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    f[0] = x.x; f[1] = x.y; f[2] = x.z; f[3] = x.w;
  } else {
    const float2 x = *reinterpret_cast<const float2*>(p);
    f[0] = x.x; f[1] = x.y;
  }
}
template <int V>
__device__ __forceinline__ void dr_load_v(const __nv_bfloat16* p, float (&f)[V]) {
  if constexpr (V == 4) {
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(x.x), b = unpack_bf16x2(x.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
    const float2 a = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p));
    f[0] = a.x; f[1] = a.y;
  }
}
template <int V>
__device__ __forceinline__ void dr_store_v(float* p, const float (&f)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  else *reinterpret_cast<float2*>(p) = make_float2(f[0], f[1]);
}
template <int V>
__device__ __forceinline__ void dr_store_v(__nv_bfloat16* p, const float (&f)[V]) {
  if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  else *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(f[0], f[1]);
}
// Activations of projections may be as exact as their storage: bf16 results take the fast exponential.
template <typename T>
__device__ __forceinline__ float dr_act(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-z));
  return dr_silu(z);
}

// Convolution of V adjacent channels of one projection, token after token, its last inputs in registers.
template <typename T, int V>
struct ConvLine {
  static constexpr int TAPS = 4;
  float w[TAPS][V], past[TAPS - 1][V];
  const T* x;

  __device__ __forceinline__ void start(const DeltaIn& a, const void* proj, int col, const T* ring, int c, int pos, const int4& seg, bool on) {
    const int taps = a.taps, C = 2 * a.G * a.D + a.H * a.DV;
    const T* conv = reinterpret_cast<const T*>(a.conv) + static_cast<long>(c) * taps;
    x = reinterpret_cast<const T*>(proj) + col;
#pragma unroll
    for (int s = 0; s < TAPS; ++s) {
      const int at = pos - s;
#pragma unroll
      for (int i = 0; i < V; ++i) {
        w[s][i] = (on && s < taps) ? dr_load(conv + i * taps + taps - 1 - s) : 0.f;
        if (s > 0) past[s > 0 ? s - 1 : 0][i] = 0.f;
      }
      if (s > 0 && on && s < taps && at >= 0)
        dr_load_v<V>(at >= seg.z ? x + (static_cast<long>(seg.x) + at - seg.z) * a.pitch : ring + static_cast<long>(at % taps) * C + c,
                     past[s > 0 ? s - 1 : 0]);
    }
  }
  __device__ __forceinline__ void next(const DeltaIn& a, long row, bool on, float (&y)[V]) {
    float cur[V];
#pragma unroll
    for (int i = 0; i < V; ++i) cur[i] = 0.f;
    if (on) dr_load_v<V>(x + row * a.pitch, cur);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      float t = w[0][i] * cur[i];
#pragma unroll
      for (int s = 1; s < TAPS; ++s) t = fmaf(w[s][i], past[s - 1][i], t);
      y[i] = dr_act<T>(t);
#pragma unroll
      for (int s = TAPS - 2; s > 0; --s) past[s][i] = past[s - 1][i];
      past[0][i] = cur[i];
    }
  }
};

// The usual sizes: heads of at most 32 V channels, at most 4 taps, everything aligned for V-wide accesses.
template <typename T, int V>
__global__ void __launch_bounds__(128)
delta_prep_wide_kernel(const __grid_constant__ DeltaIn a, const int4* __restrict__ runs, const int4* __restrict__ segs,
                       float* __restrict__ q_out, float* __restrict__ k_out, float* __restrict__ v_out, float* __restrict__ g_out,
                       float* __restrict__ beta_out, float* __restrict__ qk_out) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, vec = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (vec >= a.G + 2 * a.H) return;
  const int4 run = runs[blockIdx.x], seg = segs[run.w];
  const int H = a.H, G = a.G, D = a.D, DV = a.DV, d = lane * V;
  const T* ring = reinterpret_cast<const T*>(a.ring) + static_cast<long>(seg.w) * a.taps * (2 * G * D + H * DV);
  if (vec < G) {
    const bool on = d < D;
    ConvLine<T, V> lq, lk;
    lq.start(a, a.q, vec * D + d, ring, vec * D + d, run.z, seg, on);
    lk.start(a, a.k, vec * D + d, ring, (G + vec) * D + d, run.z, seg, on);
    const float dim = 1.f / sqrtf(static_cast<float>(D));
    for (int i = 0; i < run.y; ++i) {
      const long row = run.x + i;
      float q[V], k[V], qq = 0.f, kk = 0.f, qk = 0.f;
      lq.next(a, row, on, q);
      lk.next(a, row, on, k);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        qq = fmaf(q[j], q[j], qq);
        kk = fmaf(k[j], k[j], kk);
        qk = fmaf(q[j], k[j], qk);
      }
      const float rq = dim / sqrtf(warp_sum(qq) + 1e-6f), rk = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
      qk = warp_sum(qk) * rq * rk;
#pragma unroll
      for (int j = 0; j < V; ++j) {
        q[j] *= rq;
        k[j] *= rk;
      }
      if (on) {
        dr_store_v<V>(q_out + (row * G + vec) * D + d, q);
        dr_store_v<V>(k_out + (row * G + vec) * D + d, k);
      }
      if (lane == 0) qk_out[row * G + vec] = qk;
    }
  } else if (vec < G + H) {
    const int h = vec - G;
    const bool on = d < DV;
    ConvLine<T, V> lv;
    lv.start(a, a.v, h * DV + d, ring, 2 * G * D + h * DV + d, run.z, seg, on);
    if (lane < run.y) beta_out[(run.x + lane) * H + h] = dr_sigmoid(dr_load(reinterpret_cast<const T*>(a.b) + (static_cast<long>(run.x) + lane) * a.b_pitch + h));
    for (int i = 0; i < run.y; ++i) {
      const long row = run.x + i;
      float v[V];
      lv.next(a, row, on, v);
      if (on) dr_store_v<V>(v_out + (row * H + h) * DV + d, v);
    }
  } else {
    const int h = vec - G - H;
    const float rate = expf(a.A_log[h]);
    const T* ap = reinterpret_cast<const T*>(a.a);
    if (!a.per_channel) {
      const long row = run.x + lane;
      if (lane < run.y) g_out[row * H + h] = dr_decay(rate, dr_load(ap + row * a.a_pitch + h) + a.dt_bias[h]);
    } else if (d < D) {
      float bias[V];
      dr_load_v<V>(a.dt_bias + h * D + d, bias);
      for (int i = 0; i < run.y; ++i) {
        const long row = run.x + i;
        float z[V];
        dr_load_v<V>(ap + row * a.a_pitch + h * D + d, z);
#pragma unroll
        for (int j = 0; j < V; ++j) z[j] = dr_decay(rate, z[j] + bias[j]);
        dr_store_v<V>(g_out + (row * H + h) * D + d, z);
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ recurrence over rows
// A warp holds 4 CPT columns of S: lane = column group (4) x row group (8); a lane has CPT columns and the rows
// {4 rg + 32 j + 0..3}. Both products with S are taken before u is known (o = (g S)^T q + u (k.q)), so a token costs one
// round of shuffles. q, k, g, v of the next tokens are copied to shared memory while the current ones are processed. More columns
// per lane mean fewer reads of q, k, g from shared memory (the bound of a full machine), fewer mean more warps (few requests).
constexpr int DS_TOK = 8;     // tokens per copy
constexpr int DS_STAGES = 4;  // copies in flight or in use: three chunks ahead cover the memory's latency

__device__ __forceinline__ void ds_copy16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ds_copy4(void* dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ds_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void ds_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ float2 ds_fma2(float2 a, float2 b, float2 c) {
  union { float2 f; unsigned long long u; } x{a}, y{b}, z{c}, r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r.u) : "l"(x.u), "l"(y.u), "l"(z.u));
  return r.f;
}
__device__ __forceinline__ float2 ds_mul2(float2 a, float2 b) {
  union { float2 f; unsigned long long u; } x{a}, y{b}, r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r.u) : "l"(x.u), "l"(y.u));
  return r.f;
}
// Row `src` of a [.., n] array into shared memory by one warp.
__device__ __forceinline__ void ds_copy_row(float* dst, const float* src, int n, int lane, bool vec) {
  if (vec) {
    for (int d = lane * 4; d < n; d += 128) ds_copy16(dst + d, src + d);
  } else {
    for (int d = lane; d < n; d += 32) ds_copy4(dst + d, src + d);
  }
}

// NR: rows per lane (multiple of 4; 8 NR >= D). Columns of a CTA: 4 CPT per warp.
template <int NR>
struct DsSmem {
  static constexpr int W = 8 * NR;  // padded width of a key
  static __host__ __device__ int stage_floats(int cols, bool per_channel) { return DS_TOK * (W * (per_channel ? 3 : 2) + cols + 4); }
};

template <typename T, int NR, int CPT, bool PC>
__global__ void __launch_bounds__(CPT == 4 ? 128 : 256, CPT == 4 ? 4 : 1)
delta_scan_kernel(const __grid_constant__ DeltaIn a, const int4* __restrict__ segs, const float* __restrict__ q, const float* __restrict__ k,
                  const float* __restrict__ v, const float* __restrict__ g, const float* __restrict__ beta, const float* __restrict__ qk,
                  float* __restrict__ out) {
  constexpr int W = DsSmem<NR>::W;
  extern __shared__ __align__(16) float ds_smem[];
  const int nwarp = blockDim.x / 32, cols = nwarp * 4 * CPT;
  const int H = a.H, G = a.G, D = a.D, DV = a.DV;
  const int h = blockIdx.y, kh = h / (H / G), c0 = blockIdx.x * cols;
  const int stage = DsSmem<NR>::stage_floats(cols, PC);
  for (int i = threadIdx.x; i < DS_STAGES * stage; i += blockDim.x) ds_smem[i] = 0.f;  // padding of keys and columns stays zero
  __syncthreads();
  pdl_wait();
  pdl_launch_dependents();
  const int4 seg = segs[blockIdx.z];  // first row, tokens, first position, state slot
  const int n = seg.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rg = lane & 7, cg = lane >> 3;
  const int col = warp * 4 * CPT + cg * CPT;  // of this CTA
  const int ncol = min(cols, DV - c0);
  float* S_mem = a.state + (static_cast<long>(seg.w) * H + h) * D * DV + c0;

  float2 S[CPT][NR / 2];
#pragma unroll
  for (int j = 0; j < NR / 2; ++j) {
    const int r = rg * 4 + (j >> 1) * 32 + (j & 1) * 2;
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
      S[c][j] = make_float2(0.f, 0.f);
      if (seg.z > 0 && col + c < ncol) {
        if (r < D) S[c][j].x = S_mem[static_cast<long>(r) * DV + col + c];
        if (r + 1 < D) S[c][j].y = S_mem[static_cast<long>(r + 1) * DV + col + c];
      }
    }
  }

  // stage layout: k [TOK][W], q [TOK][W], (g [TOK][W],) v [TOK][cols], beta, q.k, g, - [TOK][4]
  constexpr int SQ = DS_TOK * W, SG = 2 * DS_TOK * W, SV = (PC ? 3 : 2) * DS_TOK * W;
  const int SC = SV + DS_TOK * cols;
  const bool vec4 = D % 4 == 0, v4 = DV % 4 == 0;
  auto fetch = [&](int t0, int buf) {
    float* base = ds_smem + buf * stage;
    const int cnt = min(DS_TOK, n - t0);
    for (int t = warp; t < cnt; t += nwarp) {
      const long row = seg.x + t0 + t;
      ds_copy_row(base + t * W, k + (row * G + kh) * D, D, lane, vec4);
      ds_copy_row(base + SQ + t * W, q + (row * G + kh) * D, D, lane, vec4);
      if (PC) ds_copy_row(base + SG + t * W, g + (row * H + h) * D, D, lane, vec4);
      ds_copy_row(base + SV + t * cols, v + (row * H + h) * DV + c0, ncol, lane, v4);
      if (lane == 0) ds_copy4(base + SC + t * 4, beta + row * H + h);
      if (lane == 1) ds_copy4(base + SC + t * 4 + 1, qk + row * G + kh);
      if (!PC && lane == 2) ds_copy4(base + SC + t * 4 + 2, g + row * H + h);
    }
    ds_commit();
  };

  const float* base = ds_smem;
  float* orow = out + (static_cast<long>(seg.x) * H + h) * DV + c0;
  auto token = [&](int t) {
    const float4 scal = *reinterpret_cast<const float4*>(base + SC + t * 4);  // beta, q.k, decay of the head
    float vv[CPT];
    dr_load_v<CPT>(base + SV + t * cols + col, vv);
    float2 kr[NR / 2], dk[CPT], dq[CPT], dk2[CPT], dq2[CPT];
    constexpr bool TWO = CPT == 2;  // two chains per sum where a lane has few columns
#pragma unroll
    for (int c = 0; c < CPT; ++c) dk[c] = dq[c] = dk2[c] = dq2[c] = make_float2(0.f, 0.f);
#pragma unroll
    for (int j = 0; j < NR / 4; ++j) {
      const int r = rg * 4 + j * 32;
      const float4 k4 = *reinterpret_cast<const float4*>(base + t * W + r);
      const float4 q4 = *reinterpret_cast<const float4*>(base + SQ + t * W + r);
      const float4 g4 = PC ? *reinterpret_cast<const float4*>(base + SG + t * W + r) : make_float4(scal.z, scal.z, scal.z, scal.z);
      kr[2 * j] = make_float2(k4.x, k4.y);
      kr[2 * j + 1] = make_float2(k4.z, k4.w);
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        S[c][2 * j] = ds_mul2(S[c][2 * j], make_float2(g4.x, g4.y));
        S[c][2 * j + 1] = ds_mul2(S[c][2 * j + 1], make_float2(g4.z, g4.w));
        dk[c] = ds_fma2(S[c][2 * j], kr[2 * j], dk[c]);
        dq[c] = ds_fma2(S[c][2 * j], make_float2(q4.x, q4.y), dq[c]);
        float2 &k_sum = TWO ? dk2[c] : dk[c], &q_sum = TWO ? dq2[c] : dq[c];
        k_sum = ds_fma2(S[c][2 * j + 1], kr[2 * j + 1], k_sum);
        q_sum = ds_fma2(S[c][2 * j + 1], make_float2(q4.z, q4.w), q_sum);
      }
    }
    // Sums over the 8 row groups.
    float x[2 * CPT];  // [product][column]
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
      x[c] = (dk[c].x + dk2[c].x) + (dk[c].y + dk2[c].y);
      x[CPT + c] = (dq[c].x + dq2[c].x) + (dq[c].y + dq2[c].y);
    }
    float u[CPT];
    if constexpr (CPT == 2) {
      // Few warps: the time of a token counts. Every lane adds up the key's sums completely, so that nothing has to travel back
      // before the write; the query's follow behind it (lane bit 0 keeps the column it names).
#pragma unroll
      for (int b = 1; b < 8; b <<= 1) {
        x[0] += __shfl_xor_sync(0xffffffffu, x[0], b);
        x[1] += __shfl_xor_sync(0xffffffffu, x[1], b);
      }
      u[0] = scal.x * (vv[0] - x[0]);
      u[1] = scal.x * (vv[1] - x[1]);
      const bool up = rg & 1;
      float y = (up ? x[3] : x[2]) + __shfl_xor_sync(0xffffffffu, up ? x[2] : x[3], 1);
      y += __shfl_xor_sync(0xffffffffu, y, 2);
      y += __shfl_xor_sync(0xffffffffu, y, 4);
      if (rg < 2 && col + rg < ncol) orow[col + rg] = fmaf(up ? u[1] : u[0], scal.y, y);
    } else {
      // Many warps: the number of shuffles counts. In every round a lane keeps half of its sums and trades the other half: by the
      // two bits of the column, then by the product; u comes back by shuffles.
      const bool b0 = rg & 1, b1 = rg & 2, b2 = rg & 4;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float keep = b0 ? x[2 * i + 1] : x[2 * i], give = b0 ? x[2 * i] : x[2 * i + 1];
        x[i] = keep + __shfl_xor_sync(0xffffffffu, give, 1);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float keep = b1 ? x[2 * i + 1] : x[2 * i], give = b1 ? x[2 * i] : x[2 * i + 1];
        x[i] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
      }
      const float y = (b2 ? x[1] : x[0]) + __shfl_xor_sync(0xffffffffu, b2 ? x[0] : x[1], 4);
      const float key_sum = __shfl_sync(0xffffffffu, y, lane & ~4);
      const float v_own = b1 ? (b0 ? vv[3] : vv[2]) : (b0 ? vv[1] : vv[0]);
      const float u_own = scal.x * (v_own - key_sum);
#pragma unroll
      for (int c = 0; c < CPT; ++c) u[c] = __shfl_sync(0xffffffffu, u_own, (lane & ~7) | c);
      if (b2 && col + (rg & 3) < ncol) orow[col + (rg & 3)] = fmaf(u_own, scal.y, y);
    }
#pragma unroll
    for (int j = 0; j < NR / 2; ++j)
#pragma unroll
      for (int c = 0; c < CPT; ++c) S[c][j] = ds_fma2(kr[j], make_float2(u[c], u[c]), S[c][j]);
    orow += static_cast<long>(H) * DV;
  };

  const int chunks = (n + DS_TOK - 1) / DS_TOK;
#pragma unroll
  for (int i = 0; i < DS_STAGES - 1; ++i) {
    if (i < chunks) fetch(i * DS_TOK, i);
    else ds_commit();
  }
  for (int ch = 0; ch < chunks; ++ch) {
    ds_wait<DS_STAGES - 2>();
    __syncthreads();  // this chunk has arrived for everyone, and everyone is done with the previous one
    const int next = ch + DS_STAGES - 1;
    if (next < chunks) fetch(next * DS_TOK, next % DS_STAGES);
    else ds_commit();
    base = ds_smem + (ch % DS_STAGES) * stage;
    const int cnt = min(DS_TOK, n - ch * DS_TOK);
    if (cnt == DS_TOK) {
#pragma unroll(CPT == 2 ? 2 : 1)
      for (int t = 0; t < DS_TOK; ++t) token(t);
    } else {
      for (int t = 0; t < cnt; ++t) token(t);
    }
  }

#pragma unroll
  for (int j = 0; j < NR / 2; ++j) {
    const int r = rg * 4 + (j >> 1) * 32 + (j & 1) * 2;
#pragma unroll
    for (int c = 0; c < CPT; ++c)
      if (col + c < ncol) {
        if (r < D) S_mem[static_cast<long>(r) * DV + col + c] = S[c][j].x;
        if (r + 1 < D) S_mem[static_cast<long>(r + 1) * DV + col + c] = S[c][j].y;
      }
  }
  // the last taps - 1 inputs of the convolution stay with the slot (sb_delta_prep has read the older ones by now)
  const int taps = a.taps, C = 2 * G * D + H * DV, keep = min(n, taps - 1);
  T* ring = reinterpret_cast<T*>(a.ring) + static_cast<long>(seg.w) * taps * C;
  const int ctas = gridDim.x * gridDim.y, cta = blockIdx.y * gridDim.x + blockIdx.x;
  for (long i = static_cast<long>(cta) * blockDim.x + threadIdx.x; i < static_cast<long>(keep) * C; i += static_cast<long>(ctas) * blockDim.x) {
    const int back = static_cast<int>(i / C), c = static_cast<int>(i - static_cast<long>(back) * C);
    const T* x = reinterpret_cast<const T*>(c < G * D ? a.q : c < 2 * G * D ? a.k : a.v);
    const int cx = c < G * D ? c : c < 2 * G * D ? c - G * D : c - 2 * G * D;
    const int at = seg.z + n - 1 - back;
    ring[static_cast<long>(at % taps) * C + c] = x[(static_cast<long>(seg.x) + n - 1 - back) * a.pitch + cx];
  }
}

// ------------------------------------------------------------------------------------------------ norm and gate of a head
__device__ __forceinline__ float dr_gate(float z, int sigmoid) { return sigmoid ? dr_sigmoid(z) : dr_silu(z); }

// One warp per (token, head): out = scale * o / rms(o) * w * gate(z)
template <typename T>
__global__ void __launch_bounds__(128)
head_gate_kernel(const float* __restrict__ o, const T* __restrict__ z, const T* __restrict__ w, T* __restrict__ out, long pairs, int H, int DV,
                 long z_pitch, long out_pitch, float eps, float scale, int sigmoid) {
  pdl_wait();
  pdl_launch_dependents();
  const long p = static_cast<long>(blockIdx.x) * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (p >= pairs) return;
  const long t = p / H;
  const int h = static_cast<int>(p - t * H);
  float x[DR_MAX / 32], ss = 0.f;
#pragma unroll
  for (int j = 0; j < DR_MAX / 32; ++j) {
    const int d = lane + 32 * j;
    x[j] = d < DV ? o[p * DV + d] : 0.f;
    ss = fmaf(x[j], x[j], ss);
  }
  const float r = scale / sqrtf(warp_sum(ss) / DV + eps);
#pragma unroll
  for (int j = 0; j < DR_MAX / 32; ++j) {
    const int d = lane + 32 * j;
    if (d < DV) dr_store(out + t * out_pitch + h * DV + d, x[j] * r * dr_load(w + d) * dr_gate(dr_load(z + t * z_pitch + h * DV + d), sigmoid));
  }
}

// The same with V adjacent columns per lane (DV <= 32 V).
template <typename T, int V>
__global__ void __launch_bounds__(128)
head_gate_wide_kernel(const float* __restrict__ o, const T* __restrict__ z, const T* __restrict__ w, T* __restrict__ out, long pairs, int H,
                      int DV, long z_pitch, long out_pitch, float eps, float scale, int sigmoid) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, d = lane * V;
  const long stride = static_cast<long>(gridDim.x) * 4;
  const bool on = d < DV;
  float wt[V], x[V], gate[V];
#pragma unroll
  for (int i = 0; i < V; ++i) wt[i] = x[i] = gate[i] = 0.f;
  if (on) dr_load_v<V>(w + d, wt);
  for (long p = static_cast<long>(blockIdx.x) * 4 + (threadIdx.x >> 5); p < pairs; p += stride) {
    const long t = p / H;
    const int h = static_cast<int>(p - t * H);
    float ss = 0.f;
    if (on) {
      dr_load_v<V>(o + p * DV + d, x);
      dr_load_v<V>(z + t * z_pitch + h * DV + d, gate);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) ss = fmaf(x[i], x[i], ss);
    const float r = scale / sqrtf(warp_sum(ss) / DV + eps);
    if (on) {
      float y[V];
#pragma unroll
      for (int i = 0; i < V; ++i) {
        float f;
        if constexpr (sizeof(T) == 2) f = __fdividef(sigmoid ? 1.f : gate[i], 1.f + __expf(-gate[i]));
        else f = dr_gate(gate[i], sigmoid);
        y[i] = x[i] * r * wt[i] * f;
      }
      dr_store_v<V>(out + t * out_pitch + h * DV + d, y);
    }
  }
}

// ------------------------------------------------------------------------------------------------ one token per request
// One CTA per (row, head), 8 warps; warp w holds rows w, w + 8, ... of S, a lane VEC adjacent columns. The state of the fast
// form stays in registers between the two uses (NR rows per warp); NR = 0 reads it twice.
struct DeltaStep {
  DeltaIn in;
  const int *slot, *active, *pos;  // state slot, whether the row counts, position of its token
  const void *z, *w;               // gate [B, H DV] (rows z_pitch apart), norm weight [DV]
  void* out;                       // [B, H DV], rows out_pitch apart
  long z_pitch, out_pitch;
  float eps, scale;
  int sigmoid;
};

template <typename T, int NR, int VEC>
__global__ void __launch_bounds__(256) delta_step_kernel(const __grid_constant__ DeltaStep s) {
  constexpr int MAXV = DR_MAX;
  __shared__ float sq[DR_MAX], sk[DR_MAX], sg[DR_MAX], sv[MAXV], red[32];
  __shared__ __align__(16) float pk[8][MAXV], pq[8][MAXV];
  const DeltaIn& a = s.in;
  const int b = blockIdx.x, h = blockIdx.y, H = a.H, G = a.G, D = a.D, DV = a.DV, taps = a.taps;
  const int kh = h / (H / G), C = 2 * G * D + H * DV;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_wait();
  pdl_launch_dependents();
  T* out = reinterpret_cast<T*>(s.out) + static_cast<long>(b) * s.out_pitch + h * DV;
  const int slot = s.slot[b];
  if (!s.active[b] || slot < 0) {  // an idle row: no state of its own to touch
    for (int d = tid; d < DV; d += 256) dr_store(out + d, 0.f);
    return;
  }
  const int pos = s.pos[b];
  float* S_mem = a.state + (static_cast<long>(slot) * H + h) * D * DV;
  const int col = lane * VEC;
  float S[NR > 0 ? NR : 1][VEC];
  if constexpr (NR > 0) {
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int r = warp + 8 * j;
#pragma unroll
      for (int c = 0; c < VEC; ++c) S[j][c] = 0.f;
      if (r < D && col < DV && pos > 0) {
        if constexpr (VEC == 4) {
          const float4 x = *reinterpret_cast<const float4*>(S_mem + static_cast<long>(r) * DV + col);
          S[j][0] = x.x; S[j][1] = x.y; S[j][2] = x.z; S[j][3] = x.w;
        } else {
          S[j][0] = S_mem[static_cast<long>(r) * DV + col];
        }
      }
    }
  }
  // convolution of this head's channels; the heads that share a query / key head all compute it, the first one keeps the input
  const T* conv = reinterpret_cast<const T*>(a.conv);
  T* ring = reinterpret_cast<T*>(a.ring) + static_cast<long>(slot) * taps * C;
  auto conv_one = [&](const T* x, int col_, int c, bool keep) {
    const T cur = x[static_cast<long>(b) * a.pitch + col_];
    float y = dr_load(conv + static_cast<long>(c) * taps + taps - 1) * dr_load(&cur);
    for (int i = 1; i < taps; ++i)
      if (pos >= i) y = fmaf(dr_load(conv + static_cast<long>(c) * taps + taps - 1 - i), dr_load(ring + static_cast<long>((pos - i) % taps) * C + c), y);
    if (keep) ring[static_cast<long>(pos % taps) * C + c] = cur;
    return dr_silu(y);
  };
  const bool first = h % (H / G) == 0;
  float qq = 0.f, kk = 0.f, qk = 0.f;
  for (int d = tid; d < D; d += 256) {
    const float q = conv_one(reinterpret_cast<const T*>(a.q), kh * D + d, kh * D + d, first);
    const float k = conv_one(reinterpret_cast<const T*>(a.k), kh * D + d, (G + kh) * D + d, first);
    qq = fmaf(q, q, qq);
    kk = fmaf(k, k, kk);
    qk = fmaf(q, k, qk);
    sq[d] = q;
    sk[d] = k;
    const T* ap = reinterpret_cast<const T*>(a.a) + static_cast<long>(b) * a.a_pitch;
    sg[d] = a.per_channel ? dr_decay(expf(a.A_log[h]), dr_load(ap + h * D + d) + a.dt_bias[h * D + d])
                          : dr_decay(expf(a.A_log[h]), dr_load(ap + h) + a.dt_bias[h]);
  }
  // the other half of the threads takes the values where the heads are narrow enough
  const int v0 = D <= 128 ? (tid + 128) & 255 : tid;
  for (int d = v0; d < DV; d += 256) sv[d] = conv_one(reinterpret_cast<const T*>(a.v), h * DV + d, 2 * G * D + h * DV + d, true);
  const float beta = dr_sigmoid(dr_load(reinterpret_cast<const T*>(a.b) + static_cast<long>(b) * a.b_pitch + h));
  qq = warp_sum(qq);
  kk = warp_sum(kk);
  qk = warp_sum(qk);
  if (lane == 0) {
    red[warp] = qq;
    red[8 + warp] = kk;
    red[16 + warp] = qk;
  }
  __syncthreads();
  qq = kk = qk = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    qq += red[i];
    kk += red[8 + i];
    qk += red[16 + i];
  }
  const float rq = 1.f / sqrtf(qq + 1e-6f) / sqrtf(static_cast<float>(D)), rk = 1.f / sqrtf(kk + 1e-6f);
  qk *= rq * rk;

  for (int c0 = col; c0 < (NR > 0 ? col + 1 : DV); c0 += 32 * VEC) {
    float dk[VEC], dq[VEC];
#pragma unroll
    for (int c = 0; c < VEC; ++c) dk[c] = dq[c] = 0.f;
    if constexpr (NR > 0) {
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        const int r = warp + 8 * j;
        if (r < D) {
          const float kr = sk[r] * rk, qr = sq[r] * rq, gr = sg[r];
#pragma unroll
          for (int c = 0; c < VEC; ++c) {
            S[j][c] *= gr;
            dk[c] = fmaf(S[j][c], kr, dk[c]);
            dq[c] = fmaf(S[j][c], qr, dq[c]);
          }
        }
      }
    } else {
      if (pos > 0)
        for (int r = warp; r < D; r += 8)
#pragma unroll
          for (int c = 0; c < VEC; ++c) {
            const float x = S_mem[static_cast<long>(r) * DV + c0 + c] * sg[r];
            dk[c] = fmaf(x, sk[r] * rk, dk[c]);
            dq[c] = fmaf(x, sq[r] * rq, dq[c]);
          }
    }
    if (c0 < DV)
#pragma unroll
      for (int c = 0; c < VEC; ++c) {
        pk[warp][c0 + c] = dk[c];
        pq[warp][c0 + c] = dq[c];
      }
  }
  __syncthreads();
  float ss = 0.f, o_keep[VEC];
  for (int c0 = col; c0 < (NR > 0 ? col + 1 : DV); c0 += 32 * VEC) {
    if (c0 >= DV) break;
    float u[VEC];
#pragma unroll
    for (int c = 0; c < VEC; ++c) {
      float x = 0.f, y = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        x += pk[i][c0 + c];
        y += pq[i][c0 + c];
      }
      u[c] = beta * (sv[c0 + c] - x);
      const float o = fmaf(u[c], qk, y);
      o_keep[c] = o;
      if (warp == 0) ss = fmaf(o, o, ss);
    }
    if constexpr (NR > 0) {
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        const int r = warp + 8 * j;
        if (r < D) {
          const float kr = sk[r] * rk;
#pragma unroll
          for (int c = 0; c < VEC; ++c) S[j][c] = fmaf(kr, u[c], S[j][c]);
          if constexpr (VEC == 4)
            *reinterpret_cast<float4*>(S_mem + static_cast<long>(r) * DV + col) = make_float4(S[j][0], S[j][1], S[j][2], S[j][3]);
          else
            S_mem[static_cast<long>(r) * DV + col] = S[j][0];
        }
      }
    } else {
      for (int r = warp; r < D; r += 8)
#pragma unroll
        for (int c = 0; c < VEC; ++c) {
          float* p = S_mem + static_cast<long>(r) * DV + c0 + c;
          *p = fmaf(sk[r] * rk, u[c], pos > 0 ? *p * sg[r] : 0.f);
        }
      if (warp == 0) sq[c0] = o_keep[0];  // (VEC is 1 here; q is not needed any more) read back below by the same thread
    }
  }
  if (warp != 0) return;
  const float r = s.scale / sqrtf(warp_sum(ss) / DV + s.eps);
  const T* z = reinterpret_cast<const T*>(s.z) + static_cast<long>(b) * s.z_pitch + h * DV;
  const T* w = reinterpret_cast<const T*>(s.w);
  for (int c0 = col; c0 < (NR > 0 ? col + 1 : DV); c0 += 32 * VEC) {
    if (c0 >= DV) break;
#pragma unroll
    for (int c = 0; c < VEC; ++c) {
      const float o = NR > 0 ? o_keep[c] : sq[c0 + c];
      dr_store(out + c0 + c, o * r * dr_load(w + c0 + c) * dr_gate(dr_load(z + c0 + c), s.sigmoid));
    }
  }
}

static int dr_check(int H, int G, int D, int DV, int taps) {
  return H <= 0 || G <= 0 || H % G != 0 || D <= 0 || DV <= 0 || D > DR_MAX || DV > DR_MAX || taps < 1 || taps > DR_MAX_TAPS;
}

template <typename... P>
static bool dr_aligned(int bytes, P... p) {
  return ((reinterpret_cast<uintptr_t>(p) | ... | uintptr_t(0)) % bytes) == 0;
}

template <typename T>
static int launch_prep(const DeltaIn& a, int nruns, const int* runs, const int* segs, float* q, float* k, float* v, float* g, float* beta,
                       float* qk, cudaStream_t s) {
  const dim3 grid(nruns, (a.G + 2 * a.H + 3) / 4);
  const int widest = a.D > a.DV ? a.D : a.DV, V = widest <= 64 ? 2 : 4;
  const bool wide = widest <= 32 * V && a.taps <= 4 && a.D % V == 0 && a.DV % V == 0 && a.pitch % V == 0 && a.a_pitch % V == 0 &&
                    dr_aligned(V * static_cast<int>(sizeof(T)), a.q, a.k, a.v, a.ring, a.per_channel ? a.a : nullptr) &&
                    dr_aligned(V * 4, q, k, v, g, a.dt_bias);
  auto kern = !wide ? delta_prep_kernel<T> : V == 2 ? delta_prep_wide_kernel<T, 2> : delta_prep_wide_kernel<T, 4>;
  return (int)launch_pdl(kern, grid, dim3(128), 0, s, a, reinterpret_cast<const int4*>(runs), reinterpret_cast<const int4*>(segs), q, k, v, g,
                         beta, qk);
}

template <typename T>
static int launch_gate(const float* o, const T* z, const T* w, T* out, long pairs, int H, int DV, long z_pitch, long out_pitch, float eps,
                       float scale, int sigmoid, cudaStream_t s) {
  const int V = DV <= 64 ? 2 : 4;
  const bool wide = DV <= 32 * V && DV % V == 0 && z_pitch % V == 0 && out_pitch % V == 0 &&
                    dr_aligned(V * static_cast<int>(sizeof(T)), z, w, out) && dr_aligned(V * 4, o);
  const long blocks = (pairs + 3) / 4, most = 148 * 16;
  auto kern = !wide ? head_gate_kernel<T> : V == 2 ? head_gate_wide_kernel<T, 2> : head_gate_wide_kernel<T, 4>;
  return (int)launch_pdl(kern, dim3(static_cast<unsigned>(wide && blocks > most ? most : blocks)), dim3(128), 0, s, o, z, w, out, pairs, H, DV,
                         z_pitch, out_pitch, eps, scale, sigmoid);
}

template <typename T, int NR, int CPT, bool PC>
static int launch_scan(const DeltaIn& a, int nseg, int warps, const int* segs, const float* q, const float* k, const float* v, const float* g,
                       const float* beta, const float* qk, float* out, cudaStream_t s) {
  const int cols = warps * 4 * CPT;
  auto kern = delta_scan_kernel<T, NR, CPT, PC>;
  if (cudaError_t e = ensure_dynamic_smem(reinterpret_cast<const void*>(kern), DS_STAGES * DsSmem<NR>::stage_floats(64, PC) * 4); e != cudaSuccess)
    return (int)e;
  // A plain launch: CTAs that start while the previous kernel still holds most of the machine would pile up on the few SMs
  // that are free, and stay there for the whole sequence.
  kern<<<dim3((a.DV + cols - 1) / cols, a.H, nseg), warps * 32, DS_STAGES * DsSmem<NR>::stage_floats(cols, PC) * 4, s>>>(
      a, reinterpret_cast<const int4*>(segs), q, k, v, g, beta, qk, out);
  return (int)cudaGetLastError();
}

// CTAs of up to 64 columns. With enough of them to fill the machine a lane takes 4 columns, otherwise 2.
template <typename T, int NR>
static int scan_shape(const DeltaIn& a, int nseg, const int* segs, const float* q, const float* k, const float* v, const float* g,
                      const float* beta, const float* qk, float* out, cudaStream_t s) {
  const bool many = NR <= 16 && static_cast<long>(nseg) * a.H * ((a.DV + 63) / 64) > 148;
  const int cols = a.DV > 32 ? 64 : a.DV > 16 ? 32 : 16;
#define SB_SCAN(CPT, PC) return launch_scan<T, NR, CPT, PC>(a, nseg, cols / (4 * CPT), segs, q, k, v, g, beta, qk, out, s)
  if constexpr (NR <= 16) {
    if (many && a.per_channel) SB_SCAN(4, true);
    if (many) SB_SCAN(4, false);
  }
  if (a.per_channel) SB_SCAN(2, true);
  SB_SCAN(2, false);
#undef SB_SCAN
}

template <typename T>
static int scan_by_width(const DeltaIn& a, int nseg, const int* segs, const float* q, const float* k, const float* v, const float* g,
                         const float* beta, const float* qk, float* out, cudaStream_t s) {
  if (a.D <= 32) return scan_shape<T, 4>(a, nseg, segs, q, k, v, g, beta, qk, out, s);
  if (a.D <= 64) return scan_shape<T, 8>(a, nseg, segs, q, k, v, g, beta, qk, out, s);
  if (a.D <= 96) return scan_shape<T, 12>(a, nseg, segs, q, k, v, g, beta, qk, out, s);
  if (a.D <= 128) return scan_shape<T, 16>(a, nseg, segs, q, k, v, g, beta, qk, out, s);
  return scan_shape<T, 32>(a, nseg, segs, q, k, v, g, beta, qk, out, s);
}

template <typename T>
static int launch_step(const DeltaStep& a, int B, cudaStream_t s) {
  const int D = a.in.D, DV = a.in.DV;
  const dim3 grid(B, a.in.H), block(256);
  if (DV % 4 == 0 && DV > 32 && DV <= 128) {
    if (D <= 32) return (int)launch_pdl(delta_step_kernel<T, 4, 4>, grid, block, 0, s, a);
    if (D <= 64) return (int)launch_pdl(delta_step_kernel<T, 8, 4>, grid, block, 0, s, a);
    if (D <= 128) return (int)launch_pdl(delta_step_kernel<T, 16, 4>, grid, block, 0, s, a);
  }
  if (DV <= 32) {
    if (D <= 64) return (int)launch_pdl(delta_step_kernel<T, 8, 1>, grid, block, 0, s, a);
    if (D <= 128) return (int)launch_pdl(delta_step_kernel<T, 16, 1>, grid, block, 0, s, a);
  }
  return (int)launch_pdl(delta_step_kernel<T, 0, 1>, grid, block, 0, s, a);
}

}  // namespace sb

// runs: nruns x int4 (first row, tokens, first position, request); segs: one int4 per request (first row, tokens, first
// position, state slot). f32: element type of the projections, conv weights and the ring (0: bf16).
extern "C" int sb_delta_prep(const void* q, const void* k, const void* v, const void* a, const void* b, long pitch, long a_pitch,
                             long b_pitch, const void* conv, const float* A_log, const float* dt_bias, const void* ring,
                             const int* runs, const int* segs, int nruns, float* q_out, float* k_out, float* v_out, float* g_out,
                             float* beta_out, float* qk_out, int H, int G, int D, int DV, int taps, int per_channel, int f32,
                             cudaStream_t s) {
  if (nruns == 0) return 0;
  if (sb::dr_check(H, G, D, DV, taps)) return (int)cudaErrorInvalidValue;
  const sb::DeltaIn in{q, k, v, a, b, pitch, a_pitch, b_pitch, conv, A_log, dt_bias, const_cast<void*>(ring), nullptr, H, G, D, DV, taps, per_channel};
  if (f32) return sb::launch_prep<float>(in, nruns, runs, segs, q_out, k_out, v_out, g_out, beta_out, qk_out, s);
  return sb::launch_prep<__nv_bfloat16>(in, nruns, runs, segs, q_out, k_out, v_out, g_out, beta_out, qk_out, s);
}

// q_in, k_in, v_in: the projections (their last rows go to the ring); q .. qk: what sb_delta_prep wrote; out [T, H, DV].
extern "C" int sb_delta_scan(const void* q_in, const void* k_in, const void* v_in, long pitch, void* ring, float* state, const int* segs,
                             int nseg, const float* q, const float* k, const float* v, const float* g, const float* beta,
                             const float* qk, float* out, int H, int G, int D, int DV, int taps, int per_channel, int f32,
                             cudaStream_t s) {
  if (nseg == 0) return 0;
  if (sb::dr_check(H, G, D, DV, taps) || nseg > 65535 || H > 65535) return (int)cudaErrorInvalidValue;
  for (const void* p : {static_cast<const void*>(q), static_cast<const void*>(k), static_cast<const void*>(v), static_cast<const void*>(g)})
    if (reinterpret_cast<uintptr_t>(p) & 15) return (int)cudaErrorInvalidValue;
  const sb::DeltaIn in{q_in, k_in, v_in, nullptr, nullptr, pitch, 0, 0, nullptr, nullptr, nullptr, ring, state, H, G, D, DV, taps, per_channel};
  if (f32) return sb::scan_by_width<float>(in, nseg, segs, q, k, v, g, beta, qk, out, s);
  return sb::scan_by_width<__nv_bfloat16>(in, nseg, segs, q, k, v, g, beta, qk, out, s);
}

extern "C" int sb_head_gate(const float* o, const void* z, const void* w, void* out, int T, int H, int DV, long z_pitch, long out_pitch,
                            float eps, float scale, int sigmoid, int f32, cudaStream_t s) {
  if (T == 0) return 0;
  if (H <= 0 || DV <= 0 || DV > sb::DR_MAX) return (int)cudaErrorInvalidValue;
  const long pairs = static_cast<long>(T) * H;
  using bf16 = __nv_bfloat16;
  if (f32) return sb::launch_gate<float>(o, (const float*)z, (const float*)w, (float*)out, pairs, H, DV, z_pitch, out_pitch, eps, scale, sigmoid, s);
  return sb::launch_gate<bf16>(o, (const bf16*)z, (const bf16*)w, (bf16*)out, pairs, H, DV, z_pitch, out_pitch, eps, scale, sigmoid, s);
}

// One token per row: slot / active / pos [B]; rows that are not active leave every state alone and give zeros.
extern "C" int sb_delta_step(const void* q, const void* k, const void* v, const void* a, const void* b, long pitch, long a_pitch,
                             long b_pitch, const void* conv, const float* A_log, const float* dt_bias, void* ring, float* state,
                             const int* slot, const int* active, const int* pos, const void* z, const void* w, void* out,
                             long z_pitch, long out_pitch, float eps, float scale, int sigmoid, int B, int H, int G, int D, int DV,
                             int taps, int per_channel, int f32, cudaStream_t s) {
  if (B == 0) return 0;
  if (sb::dr_check(H, G, D, DV, taps) || H > 65535 || (reinterpret_cast<uintptr_t>(state) & 15)) return (int)cudaErrorInvalidValue;
  const sb::DeltaStep st{{q, k, v, a, b, pitch, a_pitch, b_pitch, conv, A_log, dt_bias, ring, state, H, G, D, DV, taps, per_channel},
                         slot, active, pos, z, w, out, z_pitch, out_pitch, eps, scale, sigmoid};
  if (f32) return sb::launch_step<float>(st, B, s);
  return sb::launch_step<__nv_bfloat16>(st, B, s);
}
