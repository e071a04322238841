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

// ------------------------------------------------------------------------------------------------ recurrence over rows
// A warp holds 8 columns of S: lane = column group (4) x row group (8); a lane has 2 columns and the rows
// {4 rg + 32 j + 0..3}. Both products with S are taken before u is known (o = (g S)^T q + u (k.q)), so a token costs one
// round of shuffles. q, k, g, v of the next tokens are copied to shared memory while the current ones are processed.
constexpr int DS_TOK = 8;  // tokens per copy

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

// NR: rows per lane (multiple of 4; 8 NR >= D). Columns of a CTA: blockDim / 4.
template <int NR>
struct DsSmem {
  static constexpr int W = 8 * NR;  // padded width of a key
  static __host__ __device__ int stage_floats(int cols, bool per_channel) { return DS_TOK * (W * (per_channel ? 3 : 2) + cols + 4); }
};

template <typename T, int NR>
__global__ void __launch_bounds__(256)
delta_scan_kernel(const __grid_constant__ DeltaIn a, const int4* __restrict__ segs, const float* __restrict__ q, const float* __restrict__ k,
                  const float* __restrict__ v, const float* __restrict__ g, const float* __restrict__ beta, const float* __restrict__ qk,
                  float* __restrict__ out) {
  constexpr int W = DsSmem<NR>::W;
  extern __shared__ __align__(16) float ds_smem[];
  const int H = a.H, G = a.G, D = a.D, DV = a.DV, cols = blockDim.x / 4;
  const int h = blockIdx.y, kh = h / (H / G), c0 = blockIdx.x * cols;
  const bool pc = a.per_channel != 0;
  const int stage = DsSmem<NR>::stage_floats(cols, pc);
  for (int i = threadIdx.x; i < 2 * stage; i += blockDim.x) ds_smem[i] = 0.f;  // padding of keys and columns stays zero
  __syncthreads();
  pdl_wait();
  pdl_launch_dependents();
  const int4 seg = segs[blockIdx.z];  // first row, tokens, first position, state slot
  const int n = seg.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rg = lane & 7, cg = lane >> 3;
  const int col = warp * 8 + cg * 2;  // of this CTA
  const int ncol = min(cols, DV - c0);
  float* S_mem = a.state + (static_cast<long>(seg.w) * H + h) * D * DV + c0;

  float2 S[2][NR / 2];
#pragma unroll
  for (int j = 0; j < NR / 2; ++j) {
    const int r = rg * 4 + (j >> 1) * 32 + (j & 1) * 2;
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      S[c][j] = make_float2(0.f, 0.f);
      if (seg.z > 0 && col + c < ncol) {
        if (r < D) S[c][j].x = S_mem[static_cast<long>(r) * DV + col + c];
        if (r + 1 < D) S[c][j].y = S_mem[static_cast<long>(r + 1) * DV + col + c];
      }
    }
  }

  // stage layout: k [TOK][W], q [TOK][W], (g [TOK][W],) v [TOK][cols], beta, q.k, g, - [TOK][4]
  const bool vec4 = D % 4 == 0, v4 = DV % 4 == 0;
  auto fetch = [&](int t0, int buf) {
    float* base = ds_smem + buf * stage;
    float *sk = base, *sq = sk + DS_TOK * W, *sg = sq + DS_TOK * W, *sv = sg + (pc ? DS_TOK * W : 0), *sc = sv + DS_TOK * cols;
    const int cnt = min(DS_TOK, n - t0);
    const long row = seg.x + t0;
    if (vec4) {
      const int w4 = D / 4;
      for (int i = threadIdx.x; i < cnt * w4; i += blockDim.x) {
        const int t = i / w4, d = (i - t * w4) * 4;
        ds_copy16(sk + t * W + d, k + ((row + t) * G + kh) * D + d);
        ds_copy16(sq + t * W + d, q + ((row + t) * G + kh) * D + d);
        if (pc) ds_copy16(sg + t * W + d, g + ((row + t) * H + h) * D + d);
      }
    } else {
      for (int i = threadIdx.x; i < cnt * D; i += blockDim.x) {
        const int t = i / D, d = i - t * D;
        ds_copy4(sk + t * W + d, k + ((row + t) * G + kh) * D + d);
        ds_copy4(sq + t * W + d, q + ((row + t) * G + kh) * D + d);
        if (pc) ds_copy4(sg + t * W + d, g + ((row + t) * H + h) * D + d);
      }
    }
    if (v4) {
      const int w4 = ncol / 4;
      for (int i = threadIdx.x; i < cnt * w4; i += blockDim.x) {
        const int t = i / w4, d = (i - t * w4) * 4;
        ds_copy16(sv + t * cols + d, v + ((row + t) * H + h) * DV + c0 + d);
      }
    } else {
      for (int i = threadIdx.x; i < cnt * ncol; i += blockDim.x) {
        const int t = i / ncol, d = i - t * ncol;
        ds_copy4(sv + t * cols + d, v + ((row + t) * H + h) * DV + c0 + d);
      }
    }
    for (int t = threadIdx.x; t < cnt; t += blockDim.x) {
      ds_copy4(sc + t * 4, beta + (row + t) * H + h);
      ds_copy4(sc + t * 4 + 1, qk + (row + t) * G + kh);
      if (!pc) ds_copy4(sc + t * 4 + 2, g + (row + t) * H + h);
    }
    ds_commit();
  };

  const int chunks = (n + DS_TOK - 1) / DS_TOK;
  fetch(0, 0);
  for (int ch = 0; ch < chunks; ++ch) {
    if (ch + 1 < chunks) {
      fetch((ch + 1) * DS_TOK, (ch + 1) & 1);
      ds_wait<1>();
    } else {
      ds_wait<0>();
    }
    __syncthreads();
    const float* base = ds_smem + (ch & 1) * stage;
    const float *sk = base, *sq = sk + DS_TOK * W, *sg = sq + DS_TOK * W, *sv = sg + (pc ? DS_TOK * W : 0), *sc = sv + DS_TOK * cols;
    const int cnt = min(DS_TOK, n - ch * DS_TOK);
    for (int t = 0; t < cnt; ++t) {
      const float4 scal = *reinterpret_cast<const float4*>(sc + t * 4);  // beta, q.k, decay of the head
      const float2 vv = *reinterpret_cast<const float2*>(sv + t * cols + col);
      float2 kr[NR / 2];
      float2 dk[2], dq[2];
      dk[0] = dk[1] = dq[0] = dq[1] = make_float2(0.f, 0.f);
#pragma unroll
      for (int j = 0; j < NR / 4; ++j) {
        const int r = rg * 4 + j * 32;
        const float4 k4 = *reinterpret_cast<const float4*>(sk + t * W + r);
        const float4 q4 = *reinterpret_cast<const float4*>(sq + t * W + r);
        const float4 g4 = pc ? *reinterpret_cast<const float4*>(sg + t * W + r) : make_float4(scal.z, scal.z, scal.z, scal.z);
        kr[2 * j] = make_float2(k4.x, k4.y);
        kr[2 * j + 1] = make_float2(k4.z, k4.w);
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          S[c][2 * j] = ds_mul2(S[c][2 * j], make_float2(g4.x, g4.y));
          S[c][2 * j + 1] = ds_mul2(S[c][2 * j + 1], make_float2(g4.z, g4.w));
          dk[c] = ds_fma2(S[c][2 * j], kr[2 * j], dk[c]);
          dq[c] = ds_fma2(S[c][2 * j], make_float2(q4.x, q4.y), dq[c]);
          dk[c] = ds_fma2(S[c][2 * j + 1], kr[2 * j + 1], dk[c]);
          dq[c] = ds_fma2(S[c][2 * j + 1], make_float2(q4.z, q4.w), dq[c]);
        }
      }
      // sums over the 8 row groups: first the two columns trade halves (lane parity picks the column it keeps) ...
      float k0 = dk[0].x + dk[0].y, k1 = dk[1].x + dk[1].y, q0 = dq[0].x + dq[0].y, q1 = dq[1].x + dq[1].y;
      const bool odd = rg & 1;
      float kx = (odd ? k1 : k0) + __shfl_xor_sync(0xffffffffu, odd ? k0 : k1, 1);
      float qx = (odd ? q1 : q0) + __shfl_xor_sync(0xffffffffu, odd ? q0 : q1, 1);
      // ... then the two products do (bit 1 of the row group: 0 keeps the key's, 1 the query's)
      const bool up = rg & 2;
      float x = (up ? qx : kx) + __shfl_xor_sync(0xffffffffu, up ? kx : qx, 2);
      x += __shfl_xor_sync(0xffffffffu, x, 4);
      // lane rg has: column rg & 1 of the key's (rg & 2 == 0) or the query's product
      const float sk_own = __shfl_sync(0xffffffffu, x, (lane & ~7) | (rg & 1));
      const float u_own = scal.x * ((odd ? vv.y : vv.x) - sk_own);
      const float u_other = __shfl_xor_sync(0xffffffffu, u_own, 1);
      const float u0 = odd ? u_other : u_own, u1 = odd ? u_own : u_other;
#pragma unroll
      for (int j = 0; j < NR / 2; ++j) {
        S[0][j] = ds_fma2(kr[j], make_float2(u0, u0), S[0][j]);
        S[1][j] = ds_fma2(kr[j], make_float2(u1, u1), S[1][j]);
      }
      if ((rg & 6) == 2 && col + (rg & 1) < ncol)
        out[((static_cast<long>(seg.x) + ch * DS_TOK + t) * H + h) * DV + c0 + col + (rg & 1)] = fmaf(u_own, scal.y, x);
    }
    __syncthreads();
  }

#pragma unroll
  for (int j = 0; j < NR / 2; ++j) {
    const int r = rg * 4 + (j >> 1) * 32 + (j & 1) * 2;
#pragma unroll
    for (int c = 0; c < 2; ++c)
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

template <typename T>
static int launch_prep(const DeltaIn& a, int nruns, const int* runs, const int* segs, float* q, float* k, float* v, float* g, float* beta,
                       float* qk, cudaStream_t s) {
  return (int)launch_pdl(delta_prep_kernel<T>, dim3(nruns, (a.G + 2 * a.H + 3) / 4), dim3(128), 0, s, a, reinterpret_cast<const int4*>(runs),
                         reinterpret_cast<const int4*>(segs), q, k, v, g, beta, qk);
}

template <typename T, int NR>
static int launch_scan(const DeltaIn& a, int nseg, const int* segs, const float* q, const float* k, const float* v, const float* g,
                       const float* beta, const float* qk, float* out, cudaStream_t s) {
  const int cols = a.DV > 32 ? 64 : a.DV > 16 ? 32 : 16;
  const int bytes = 2 * DsSmem<NR>::stage_floats(cols, a.per_channel != 0) * 4;
  auto kern = delta_scan_kernel<T, NR>;
  if (cudaError_t e = ensure_dynamic_smem(reinterpret_cast<const void*>(kern), 2 * DsSmem<NR>::stage_floats(64, true) * 4); e != cudaSuccess)
    return (int)e;
  return (int)launch_pdl(kern, dim3((a.DV + cols - 1) / cols, a.H, nseg), dim3(cols * 4), bytes, s, a, reinterpret_cast<const int4*>(segs), q, k,
                         v, g, beta, qk, out);
}

template <typename T>
static int scan_by_width(const DeltaIn& a, int nseg, const int* segs, const float* q, const float* k, const float* v, const float* g,
                         const float* beta, const float* qk, float* out, cudaStream_t s) {
  if (a.D <= 32) return launch_scan<T, 4>(a, nseg, segs, q, k, v, g, beta, qk, out, s);
  if (a.D <= 64) return launch_scan<T, 8>(a, nseg, segs, q, k, v, g, beta, qk, out, s);
  if (a.D <= 96) return launch_scan<T, 12>(a, nseg, segs, q, k, v, g, beta, qk, out, s);
  if (a.D <= 128) return launch_scan<T, 16>(a, nseg, segs, q, k, v, g, beta, qk, out, s);
  return launch_scan<T, 32>(a, nseg, segs, q, k, v, g, beta, qk, out, s);
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
  const dim3 grid(static_cast<unsigned>((pairs + 3) / 4));
  using bf16 = __nv_bfloat16;
  if (f32)
    return (int)sb::launch_pdl(sb::head_gate_kernel<float>, grid, dim3(128), 0, s, o, (const float*)z, (const float*)w, (float*)out, pairs, H, DV,
                               z_pitch, out_pitch, eps, scale, sigmoid);
  return (int)sb::launch_pdl(sb::head_gate_kernel<bf16>, grid, dim3(128), 0, s, o, (const bf16*)z, (const bf16*)w, (bf16*)out, pairs, H, DV,
                             z_pitch, out_pitch, eps, scale, sigmoid);
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
