// Linear recurrences with one decay per head and token (state-space duality of Mamba-2, matrix memory of xLSTM) over per-request
// states that live in slots. Per head, with S [D, DV] in fp32:
//
//     S <- f S + w k v^T        o = S^T q  (+ skip v)
//
//   state space   f = exp(-exp(A_log) dt), w = dt = softplus(projection + dt_bias); q, k, v = C, B, x, projections that passed a short
//                 causal convolution (with bias) and silu; head h uses C and B of group h / (H / G)
//   matrix memory log gates i, f' capped softly, m <- max(f' + m, i), f = exp(f' + m_before - m), w = exp(i - m); q times D^-1/2; a
//                 normaliser n <- f n + w k beside S; the output is divided by max(|n q|, exp(-m)) + 1e-6
//
//   sb_ssd_prep      packed rows -> fp32 x, B, C and gates of every token
//   sb_memory_prep   the same for q, k, v and the gates of the matrix memory (the running maximum is carried here)
//   sb_linear_scan   the recurrence over the rows of every request, states read and left in their slots
//   sb_ssd_step, sb_memory_step   one token per request, all of the above in one launch
//   sb_part_gate     RMS norm of parts of a row, weight and gate, bf16 / fp32 result
//
// Everything behind the projections is fp32. The normaliser is one more column of S whose v is 1: an extra CTA per head. The running
// maximum of a slot has two places, by position parity: whoever computes the next one never overwrites what others still read.
// The convolution's inputs live in a ring of `taps` rows per slot (row = position mod taps).
#include <type_traits>

#include "common.cuh"

namespace sb {

constexpr int LS_MAX_D = 512;
constexpr int LS_MAX_TAPS = 16;

__device__ __forceinline__ float ls_load(const float* p) { return *p; }
__device__ __forceinline__ float ls_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void ls_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void ls_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float ls_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float ls_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float ls_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float ls_cap(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float ls_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// V adjacent elements as floats, and back.
template <int V>
__device__ __forceinline__ void ls_load_v(const float* p, float (&f)[V]) {
  if constexpr (V == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    f[0] = x.x; f[1] = x.y; f[2] = x.z; f[3] = x.w;
  } else {
    f[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void ls_load_v(const __nv_bfloat16* p, float (&f)[V]) {
  if constexpr (V == 4) {
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(x.x), b = unpack_bf16x2(x.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
    f[0] = __bfloat162float(*p);
  }
}
template <int V>
__device__ __forceinline__ void ls_store_v(float* p, const float (&f)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  else *p = f[0];
}
template <int V>
__device__ __forceinline__ void ls_store_v(__nv_bfloat16* p, const float (&f)[V]) {
  if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  else *p = __float2bfloat16(f[0]);
}
// Activations of projections may be as exact as their storage.
template <typename T>
__device__ __forceinline__ float ls_act(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-z));
  return ls_silu(z);
}

// ------------------------------------------------------------------------------------------------ state space: inputs
// Projections of one layer, element type T; rows are `pitch` elements apart. Convolution channels in the order x, B, C.
struct SsdIn {
  const void *x, *B, *C, *dt;  // [T, H DV], [T, G D], [T, G D], [T, H]
  long pitch;
  const void *conv, *conv_b;   // [H DV + 2 G D, taps], [H DV + 2 G D]
  const float *A_log, *dt_bias;
  const void* ring;            // [slots, taps, H DV + 2 G D]
  int H, G, D, DV, taps;
};

__device__ __forceinline__ float4 ssd_gate(float z, float bias, float A_log) {
  const float dt = ls_softplus(z + bias);
  return make_float4(expf(-expf(A_log) * dt), dt, 0.f, 0.f);
}

// One thread per V adjacent channels of one projection and run of tokens; the last y-block works out the gates. V divides the widths
// of the three projections. NT: taps whose inputs a thread keeps in registers (0: any number, read again for every token).
template <typename T, int V, int NT>
__global__ void __launch_bounds__(128)
ssd_prep_kernel(const __grid_constant__ SsdIn a, const int4* __restrict__ runs, const int4* __restrict__ segs, float* __restrict__ x_out,
                float* __restrict__ B_out, float* __restrict__ C_out, float4* __restrict__ gates) {
  pdl_wait();
  pdl_launch_dependents();
  const int4 run = runs[blockIdx.x];  // first row, tokens, first position, request
  const int wx = a.H * a.DV, wb = a.G * a.D, ch = wx + 2 * wb, taps = a.taps;
  if (blockIdx.y == gridDim.y - 1) {
    for (int i = threadIdx.x; i < run.y * a.H; i += 128) {
      const int h = i % a.H;
      const long row = run.x + i / a.H;
      gates[row * a.H + h] = ssd_gate(ls_load(reinterpret_cast<const T*>(a.dt) + row * a.pitch + h), a.dt_bias[h], a.A_log[h]);
    }
    return;
  }
  const int c = (blockIdx.y * 128 + threadIdx.x) * V;
  if (c >= ch) return;
  const int4 seg = segs[run.w];  // first row, tokens, first position, state slot
  const int part = c < wx ? 0 : c < wx + wb ? 1 : 2, col = c - (part == 0 ? 0 : part == 1 ? wx : wx + wb);
  const T* src = reinterpret_cast<const T*>(part == 0 ? a.x : part == 1 ? a.B : a.C) + col;
  const long width = part == 0 ? wx : wb;
  float* dst = (part == 0 ? x_out : part == 1 ? B_out : C_out) + col;
  const T* ring = reinterpret_cast<const T*>(a.ring) + static_cast<long>(seg.w) * taps * ch + c;
  const T* conv = reinterpret_cast<const T*>(a.conv) + static_cast<long>(c) * taps;
  float bias[V];
#pragma unroll
  for (int i = 0; i < V; ++i) bias[i] = ls_load(reinterpret_cast<const T*>(a.conv_b) + c + i);
  // input at position `at`: from the pass's rows when it has the token, from the ring when an earlier pass had it, zero before
  auto input = [&](int at, float (&f)[V]) {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = 0.f;
    if (at >= seg.z) ls_load_v<V>(src + (static_cast<long>(seg.x) + at - seg.z) * a.pitch, f);
    else if (at >= 0) ls_load_v<V>(ring + static_cast<long>(at % taps) * ch, f);
  };
  if constexpr (NT > 0) {
    float w[NT][V], past[NT][V];  // past[s]: input s tokens back
#pragma unroll
    for (int s = 0; s < NT; ++s) {
#pragma unroll
      for (int i = 0; i < V; ++i) w[s][i] = s < taps ? ls_load(conv + i * taps + taps - 1 - s) : 0.f;
      if (s > 0 && s < taps) {
        input(run.z - s, past[s]);
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) past[s][i] = 0.f;
      }
    }
    for (int t = 0; t < run.y; ++t) {
      float y[V];
      ls_load_v<V>(src + (static_cast<long>(run.x) + t) * a.pitch, past[0]);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        float z = bias[i];
#pragma unroll
        for (int s = NT - 1; s >= 0; --s) z = fmaf(w[s][i], past[s][i], z);
        y[i] = ls_act<T>(z);
#pragma unroll
        for (int s = NT - 1; s > 0; --s) past[s][i] = past[s - 1][i];
      }
      ls_store_v<V>(dst + (static_cast<long>(run.x) + t) * width, y);
    }
  } else {
    for (int t = 0; t < run.y; ++t) {
      float z[V];
#pragma unroll
      for (int i = 0; i < V; ++i) z[i] = bias[i];
      for (int s = taps - 1; s >= 0; --s) {
        float f[V];
        input(run.z + t - s, f);
#pragma unroll
        for (int i = 0; i < V; ++i) z[i] = fmaf(ls_load(conv + i * taps + taps - 1 - s), f[i], z[i]);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) z[i] = ls_act<T>(z[i]);
      ls_store_v<V>(dst + (static_cast<long>(run.x) + t) * width, z);
    }
  }
}

// ------------------------------------------------------------------------------------------------ matrix memory: inputs
struct MemoryIn {
  const void *q, *k, *v, *i, *f;  // [T, H D], [T, H D], [T, H DV], [T, H], [T, H]
  long pitch;
  const float *i_b, *f_b;         // [H]
  float* top;                     // [slots, H, 2] running maximum before a position of even / odd number
  int H, D, DV;
  float cap;
};

// fp32 copies of q, k, v by most CTAs; the first `gate_ctas` carry the running maximum, one warp per (request, head), 32 tokens per
// turn by a scan of (sum of f, max) pairs: m after token t = max(F_t + m, max over s <= t of (i_s + F_t - F_s)).
template <typename T, int V>
__global__ void __launch_bounds__(256)
memory_prep_kernel(const __grid_constant__ MemoryIn a, const int4* __restrict__ segs, int nseg, int rows, int gate_ctas,
                   float* __restrict__ q_out, float* __restrict__ k_out, float* __restrict__ v_out, float4* __restrict__ gates) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, H = a.H;
  if (static_cast<int>(blockIdx.x) < gate_ctas) {
    const int job = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (job >= nseg * H) return;
    const int4 seg = segs[job / H];
    const int h = job % H;
    float* top = a.top + (static_cast<long>(seg.w) * H + h) * 2;
    float m = seg.z > 0 ? top[seg.z & 1] : 0.f;
    const T* ip = reinterpret_cast<const T*>(a.i) + static_cast<long>(seg.x) * a.pitch + h;
    const T* fp = reinterpret_cast<const T*>(a.f) + static_cast<long>(seg.x) * a.pitch + h;
    float zi = 0.f, zf = 0.f;
    if (lane < seg.y) {
      zi = ls_load(ip + lane * a.pitch);
      zf = ls_load(fp + lane * a.pitch);
    }
    for (int t0 = 0; t0 < seg.y; t0 += 32) {
      const int t = t0 + lane;
      const bool on = t < seg.y;
      const float li = ls_cap(zi + a.i_b[h], a.cap), lf = ls_log_sigmoid(ls_cap(zf + a.f_b[h], a.cap));
      if (t + 32 < seg.y) {  // the next turn's inputs
        zi = ls_load(ip + (t + 32) * a.pitch);
        zf = ls_load(fp + (t + 32) * a.pitch);
      }
      float F = on ? lf : 0.f, M = on ? li : -INFINITY;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float Fo = __shfl_up_sync(0xffffffffu, F, o), Mo = __shfl_up_sync(0xffffffffu, M, o);
        if (lane >= o) {
          M = fmaxf(M, Mo + F);
          F += Fo;
        }
      }
      const float now = fmaxf(F + m, M);
      float before = __shfl_up_sync(0xffffffffu, now, 1);
      if (lane == 0) before = m;
      if (on) gates[(static_cast<long>(seg.x) + t) * H + h] = make_float4(expf(lf + before - now), expf(li - now), expf(-now), 0.f);
      m = __shfl_sync(0xffffffffu, now, min(31, seg.y - 1 - t0));
    }
    if (lane == 0) top[(seg.z + seg.y) & 1] = m;
    return;
  }
  const int nq = H * a.D / V, nv = H * a.DV / V, per = 2 * nq + nv;
  const float unit = 1.f / sqrtf(static_cast<float>(a.D));
  const long n = static_cast<long>(rows) * per, stride = static_cast<long>(gridDim.x - gate_ctas) * 256;
  for (long e = static_cast<long>(blockIdx.x - gate_ctas) * 256 + threadIdx.x; e < n; e += stride) {
    const long t = e / per;
    const int c = static_cast<int>(e - t * per);
    float f[V];
    if (c < nq) {
      ls_load_v<V>(reinterpret_cast<const T*>(a.q) + t * a.pitch + c * V, f);
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] *= unit;
      ls_store_v<V>(q_out + (t * nq + c) * V, f);
    } else if (c < 2 * nq) {
      ls_load_v<V>(reinterpret_cast<const T*>(a.k) + t * a.pitch + (c - nq) * V, f);
      ls_store_v<V>(k_out + (t * nq + c - nq) * V, f);
    } else {
      ls_load_v<V>(reinterpret_cast<const T*>(a.v) + t * a.pitch + (c - 2 * nq) * V, f);
      ls_store_v<V>(v_out + (t * nv + c - 2 * nq) * V, f);
    }
  }
}

// ------------------------------------------------------------------------------------------------ recurrence over rows
// A warp holds (32 / RG) CPT columns of S: lane = column group x row group (RG of them); a lane has CPT columns and the rows
// {4 rg + 4 RG j + 0..3}. q, k, v and gates of the next tokens are copied to shared memory while the current ones are processed. Nothing
// that a token computes is needed by the next one but S itself, so tokens overlap; sums over the rows are taken for two
// tokens at a time.
//
// S is kept divided by the product F of the decays since the start of a chunk of 8 tokens: S' <- S' + k (w / F) v^T and o = F S'^T q cost
// two operations per element instead of three. The numbers in S' differ from those in S by a common factor only, so nothing is
// lost as long as F stays far from the end of the number range; a chunk in which it does not decays S token by token.
constexpr int LS_TOK = 8;     // tokens per copy
constexpr int LS_STAGES = 4;  // copies in flight or in use

__device__ __forceinline__ void ls_copy16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ls_copy4(void* dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ls_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void ls_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ float2 ls_fma2(float2 a, float2 b, float2 c) {
  union { float2 f; unsigned long long u; } x{a}, y{b}, z{c}, r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r.u) : "l"(x.u), "l"(y.u), "l"(z.u));
  return r.f;
}
__device__ __forceinline__ float2 ls_mul2(float2 a, float2 b) {
  union { float2 f; unsigned long long u; } x{a}, y{b}, r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r.u) : "l"(x.u), "l"(y.u));
  return r.f;
}
// A row of n floats into shared memory by one warp.
__device__ __forceinline__ void ls_copy_row(float* dst, const float* src, int n, int lane, bool vec) {
  if (vec) {
    for (int d = lane * 4; d < n; d += 128) ls_copy16(dst + d, src + d);
  } else {
    for (int d = lane; d < n; d += 32) ls_copy4(dst + d, src + d);
  }
}

struct Scan {
  const float *q, *k, *v;  // [T, G D], [T, G D], [T, H DV]
  const float4* gates;     // [T, H]: f, w, least divisor
  const float* skip;       // [H]: v's own part of the output, or null
  float* out;              // [T, H, DV]
  float* state;            // [slots, H, D, DV]
  float *norm, *den;       // [slots, H, D] normaliser and [T, H] divisors, or null
  const int4* segs;
  int H, G, D, DV, blocks;  // column blocks of a head (the next one is the normaliser)
  // ring of convolution inputs (elements of `esize` bytes): the last taps - 1 rows of every request go there
  void* ring;
  const void* in[3];       // their projections, rows `in_pitch` elements apart
  long in_pitch;
  int width[3], taps, esize;
};

constexpr float LS_LEAST = 1e-18f;  // smallest product of a chunk's decays that S is divided by

template <int RG, int NR>
struct LsSmem {
  static constexpr int W = RG * NR;  // padded width of a key
  static __host__ __device__ int stage_floats(int cols) { return LS_TOK * (2 * W + cols + 4); }
};

// Sums over the RG lanes of a row group of N values per lane: in every round a lane keeps half of its sums and trades the others, by
// the bits of its number; when one is left the rest is summed plainly. Lane rg ends up with value rg mod N (N <= RG).
template <int RG, int N>
__device__ __forceinline__ float ls_reduce(float (&x)[N], int rg) {
  int bit = 1;
#pragma unroll
  for (int n = N; n > 1; n /= 2, bit *= 2) {
    const bool up = rg & bit;
#pragma unroll
    for (int i = 0; i < n / 2; ++i) x[i] = (up ? x[2 * i + 1] : x[2 * i]) + __shfl_xor_sync(0xffffffffu, up ? x[2 * i] : x[2 * i + 1], bit);
  }
  float o = x[0];
#pragma unroll
  for (int b = N; b < RG; b *= 2) o += __shfl_xor_sync(0xffffffffu, o, b);
  return o;
}

template <int RG, int NR, int CPT, int THREADS, int CTAS>
__global__ void __launch_bounds__(THREADS, CTAS) linear_scan_kernel(const __grid_constant__ Scan a) {
  using Smem = LsSmem<RG, NR>;
  constexpr int W = Smem::W, CG = 32 / RG;
  extern __shared__ __align__(16) float ls_smem[];
  const int nwarp = blockDim.x / 32, cols = nwarp * CG * CPT;
  const int H = a.H, G = a.G, D = a.D, DV = a.DV;
  const int h = blockIdx.y, kh = h / (H / G);
  const bool is_n = static_cast<int>(blockIdx.x) == a.blocks;  // the normaliser: one column whose v is 1
  const int c0 = is_n ? 0 : blockIdx.x * cols;
  const int stage = Smem::stage_floats(cols);
  // stage layout: k [TOK][W], q [TOK][W], v [TOK][cols], gates [TOK][4]
  constexpr int SQ = LS_TOK * W, SV = 2 * LS_TOK * W;
  const int SC = SV + LS_TOK * cols;
  for (int i = threadIdx.x; i < LS_STAGES * stage; i += blockDim.x) {  // padding of keys and columns stays zero
    const int at = i % stage;
    ls_smem[i] = is_n && at >= SV && at < SC ? 1.f : 0.f;
  }
  __syncthreads();
  const int4 seg = a.segs[blockIdx.z];  // first row, tokens, first position, state slot
  const int n = seg.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rg = lane % RG, cg = lane / RG;
  const int col = (warp * CG + cg) * CPT;  // of this CTA
  const int pitch = is_n ? 1 : DV, ncol = is_n ? 1 : min(cols, DV - c0);
  const long head = static_cast<long>(seg.w) * H + h;
  float* S_mem = is_n ? a.norm + head * D : a.state + head * D * DV + c0;

  float2 S[CPT][NR / 2];
#pragma unroll
  for (int j = 0; j < NR / 2; ++j) {
    const int r = rg * 4 + (j >> 1) * (4 * RG) + (j & 1) * 2;
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
      S[c][j] = make_float2(0.f, 0.f);
      if (seg.z > 0 && col + c < ncol) {
        if (r < D) S[c][j].x = S_mem[static_cast<long>(r) * pitch + col + c];
        if (r + 1 < D) S[c][j].y = S_mem[static_cast<long>(r + 1) * pitch + col + c];
      }
    }
  }

  const bool vec4 = D % 4 == 0, v4 = DV % 4 == 0;
  auto fetch = [&](int t0, int buf) {
    float* base = ls_smem + buf * stage;
    const int cnt = min(LS_TOK, n - t0);
    for (int t = warp; t < cnt; t += nwarp) {
      const long row = seg.x + t0 + t;
      ls_copy_row(base + t * W, a.k + (row * G + kh) * D, D, lane, vec4);
      ls_copy_row(base + SQ + t * W, a.q + (row * G + kh) * D, D, lane, vec4);
      if (!is_n) ls_copy_row(base + SV + t * cols, a.v + (row * H + h) * DV + c0, ncol, lane, v4);
      if (lane == 0) ls_copy16(base + SC + t * 4, a.gates + row * H + h);
    }
    ls_commit();
  };

  const float* base = ls_smem;
  const float skip = a.skip != nullptr ? a.skip[h] : 0.f;
  float* orow = is_n ? a.den + static_cast<long>(seg.x) * H + h : a.out + (static_cast<long>(seg.x) * H + h) * DV + c0;
  const long ostep = is_n ? H : static_cast<long>(H) * DV;
  float F = 1.f;  // what S is divided by
  // one token: S and this lane's part of S^T q into o[2 c + which]. `divided`: S divided by F, or decayed token by token
  auto advance = [&](auto divided, int t, int which, float (&o)[2 * CPT]) {
    const float2 gate = *reinterpret_cast<const float2*>(base + SC + t * 4);
    float2 u2[CPT], acc[CPT];
    float w = gate.y;
    if constexpr (decltype(divided)::value) {
      F *= gate.x;
      w = __fdividef(w, F);
    } else {
      const float2 f2 = make_float2(gate.x, gate.x);
#pragma unroll
      for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int j = 0; j < NR / 2; ++j) S[c][j] = ls_mul2(S[c][j], f2);
    }
#pragma unroll
    for (int c = 0; c < CPT; c += 4) {
      const float4 v = *reinterpret_cast<const float4*>(base + SV + t * cols + col + c);
      u2[c] = make_float2(v.x * w, v.x * w);
      u2[c + 1] = make_float2(v.y * w, v.y * w);
      u2[c + 2] = make_float2(v.z * w, v.z * w);
      u2[c + 3] = make_float2(v.w * w, v.w * w);
    }
#pragma unroll
    for (int j = 0; j < NR / 4; ++j) {
      const int r = rg * 4 + j * 4 * RG;
      const float4 k4 = *reinterpret_cast<const float4*>(base + t * W + r);
      const float4 q4 = *reinterpret_cast<const float4*>(base + SQ + t * W + r);
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        S[c][2 * j] = ls_fma2(make_float2(k4.x, k4.y), u2[c], S[c][2 * j]);
        S[c][2 * j + 1] = ls_fma2(make_float2(k4.z, k4.w), u2[c], S[c][2 * j + 1]);
        acc[c] = j == 0 ? ls_mul2(S[c][0], make_float2(q4.x, q4.y)) : ls_fma2(S[c][2 * j], make_float2(q4.x, q4.y), acc[c]);
        acc[c] = ls_fma2(S[c][2 * j + 1], make_float2(q4.z, q4.w), acc[c]);
      }
    }
#pragma unroll
    for (int c = 0; c < CPT; ++c) o[2 * c + which] = acc[c].x + acc[c].y;
  };
  auto pair = [&](auto divided, int t, bool second) {
    float x[2 * CPT];
    advance(divided, t, 0, x);
    const float F0 = F;
    if (second) {
      advance(divided, t + 1, 1, x);
    } else {
#pragma unroll
      for (int c = 0; c < CPT; ++c) x[2 * c + 1] = 0.f;
    }
    const float o = ls_reduce<RG, 2 * CPT>(x, rg) * (rg & 1 ? F : F0);
    const int tok = t + (rg & 1), c = col + ((rg >> 1) & (CPT - 1));
    if (rg >= 2 * CPT || c >= ncol || ((rg & 1) && !second)) return;
    if (is_n) orow[tok * ostep] = fmaxf(fabsf(o), base[SC + tok * 4 + 2]) + 1e-6f;
    else orow[tok * ostep + c] = fmaf(skip, base[SV + tok * cols + c], o);
  };
  auto tokens = [&](auto divided, int cnt) {
    if (cnt == LS_TOK) {  // unrolled: the sums of a pair of tokens are taken underneath the next one's products
#pragma unroll 2
      for (int t = 0; t < LS_TOK; t += 2) pair(divided, t, true);
    } else {
#pragma unroll 1
      for (int t = 0; t < cnt; t += 2) pair(divided, t, t + 1 < cnt);
    }
  };

  const int chunks = (n + LS_TOK - 1) / LS_TOK;
#pragma unroll
  for (int i = 0; i < LS_STAGES - 1; ++i) {
    if (i < chunks) fetch(i * LS_TOK, i);
    else ls_commit();
  }
  for (int ch = 0; ch < chunks; ++ch) {
    ls_wait<LS_STAGES - 2>();
    __syncthreads();  // this chunk has arrived for everyone, and everyone is done with the previous one
    const int next = ch + LS_STAGES - 1;
    if (next < chunks) fetch(next * LS_TOK, next % LS_STAGES);
    else ls_commit();
    base = ls_smem + (ch % LS_STAGES) * stage;
    const int cnt = min(LS_TOK, n - ch * LS_TOK);
    F = 1.f;
    for (int t = 0; t < cnt; ++t) F *= base[SC + t * 4];
    const bool divided = F > LS_LEAST;  // the same for every thread
    F = 1.f;
    if (divided) {
      tokens(std::true_type(), cnt);
      const float2 f2 = make_float2(F, F);
#pragma unroll
      for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int j = 0; j < NR / 2; ++j) S[c][j] = ls_mul2(S[c][j], f2);
    } else {
      tokens(std::false_type(), cnt);
    }
    orow += LS_TOK * ostep;
  }

#pragma unroll
  for (int j = 0; j < NR / 2; ++j) {
    const int r = rg * 4 + (j >> 1) * (4 * RG) + (j & 1) * 2;
#pragma unroll
    for (int c = 0; c < CPT; ++c)
      if (col + c < ncol) {
        if (r < D) S_mem[static_cast<long>(r) * pitch + col + c] = S[c][j].x;
        if (r + 1 < D) S_mem[static_cast<long>(r + 1) * pitch + col + c] = S[c][j].y;
      }
  }
  if (a.ring == nullptr) return;
  // the last taps - 1 inputs of the convolution stay with the slot (sb_ssd_prep has read the older ones by now)
  const int taps = a.taps, C = a.width[0] + a.width[1] + a.width[2], keep = min(n, taps - 1);
  const int ctas = gridDim.x * gridDim.y, cta = blockIdx.y * gridDim.x + blockIdx.x;
  for (long i = static_cast<long>(cta) * blockDim.x + threadIdx.x; i < static_cast<long>(keep) * C; i += static_cast<long>(ctas) * blockDim.x) {
    const int back = static_cast<int>(i / C), c = static_cast<int>(i - static_cast<long>(back) * C);
    const int part = c < a.width[0] ? 0 : c < a.width[0] + a.width[1] ? 1 : 2;
    const int cx = c - (part == 0 ? 0 : part == 1 ? a.width[0] : a.width[0] + a.width[1]);
    const long dst = (static_cast<long>(seg.w) * taps + (seg.z + n - 1 - back) % taps) * C + c;
    const long src = (static_cast<long>(seg.x) + n - 1 - back) * a.in_pitch + cx;
    if (a.esize == 2) reinterpret_cast<uint16_t*>(a.ring)[dst] = reinterpret_cast<const uint16_t*>(a.in[part])[src];
    else reinterpret_cast<uint32_t*>(a.ring)[dst] = reinterpret_cast<const uint32_t*>(a.in[part])[src];
  }
}

// ------------------------------------------------------------------------------------------------ one token per request
// One CTA per (row, head, block of columns; the last block is the normaliser). Threads: LPR lanes of VEC adjacent columns per row of
// S, 256 / LPR rows at a time.
struct Step {
  float* state;        // [slots, H, D, DV]
  const int *slot, *active, *pos;
  float* out;          // [B, H, DV]
  int H, G, D, DV, blocks, lpr;
};
constexpr int LS_COLS = 64;

// S <- f S + w k v^T and o = S^T q over the columns [c0, c0 + ncol) of a head; su: w v by column. Returns o of column tid < ncol.
template <int VEC>
__device__ __forceinline__ float step_columns(float* S_mem, int pitch, int ncol, int D, int lpr, bool have, float f, const float* sq,
                                              const float* sk, const float* su, float* part) {
  const int tid = threadIdx.x, rows = 256 / lpr, r0 = tid / lpr, c = (tid % lpr) * VEC;
  float acc[VEC], u[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    acc[i] = 0.f;
    u[i] = c + i < ncol ? su[c + i] : 0.f;
  }
  constexpr int AHEAD = 8;
  if (c < ncol)
    for (int b = r0; b < D; b += rows * AHEAD) {
      float S[AHEAD][VEC];
#pragma unroll
      for (int j = 0; j < AHEAD; ++j) {
        const int r = b + j * rows;
#pragma unroll
        for (int i = 0; i < VEC; ++i) S[j][i] = 0.f;
        if (have && r < D) ls_load_v<VEC>(S_mem + static_cast<long>(r) * pitch + c, S[j]);
      }
#pragma unroll
      for (int j = 0; j < AHEAD; ++j) {
        const int r = b + j * rows;
        if (r < D) {
#pragma unroll
          for (int i = 0; i < VEC; ++i) {
            S[j][i] = fmaf(S[j][i], f, sk[r] * u[i]);
            acc[i] = fmaf(S[j][i], sq[r], acc[i]);
          }
          ls_store_v<VEC>(S_mem + static_cast<long>(r) * pitch + c, S[j]);
        }
      }
    }
  // sums over the row groups: part [rows][lpr * VEC]
#pragma unroll
  for (int i = 0; i < VEC; ++i) part[r0 * lpr * VEC + c + i] = acc[i];
  __syncthreads();
  float o = 0.f;
  if (tid < ncol)
    for (int r = 0; r < rows; ++r) o += part[r * lpr * VEC + tid];
  return o;
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) ssd_step_kernel(const __grid_constant__ SsdIn a, const __grid_constant__ Step s, const float* __restrict__ skip) {
  __shared__ float sq[LS_MAX_D], sk[LS_MAX_D], sx[LS_COLS], su[LS_COLS], part[256 * VEC];
  const int b = blockIdx.x, h = blockIdx.y, H = a.H, G = a.G, D = a.D, DV = a.DV, taps = a.taps, tid = threadIdx.x;
  const int kh = h / (H / G), c0 = blockIdx.z * LS_COLS, ncol = min(LS_COLS, DV - c0), C = H * DV + 2 * G * D;
  pdl_wait();
  pdl_launch_dependents();
  const int slot = s.slot[b];
  float* out = s.out + (static_cast<long>(b) * H + h) * DV + c0;
  if (!s.active[b] || slot < 0) {  // an idle row: no state of its own to touch
    if (tid < ncol) out[tid] = 0.f;
    return;
  }
  const int pos = s.pos[b];
  const T* conv = reinterpret_cast<const T*>(a.conv);
  T* ring = const_cast<T*>(reinterpret_cast<const T*>(a.ring)) + static_cast<long>(slot) * taps * C;
  auto conv_one = [&](const void* proj, int col, int c, bool keep) {
    const T cur = reinterpret_cast<const T*>(proj)[static_cast<long>(b) * a.pitch + col];
    float z = ls_load(reinterpret_cast<const T*>(a.conv_b) + c);
    for (int i = taps - 1; i > 0; --i)
      if (pos >= i) z = fmaf(ls_load(conv + static_cast<long>(c) * taps + taps - 1 - i), ls_load(ring + static_cast<long>((pos - i) % taps) * C + c), z);
    z = fmaf(ls_load(conv + static_cast<long>(c) * taps + taps - 1), ls_load(&cur), z);
    if (keep) ring[static_cast<long>(pos % taps) * C + c] = cur;
    return ls_act<T>(z);
  };
  const bool first = h % (H / G) == 0 && blockIdx.z == 0;  // the heads of a group all compute B and C, the first one keeps the input
  const float4 gate = ssd_gate(ls_load(reinterpret_cast<const T*>(a.dt) + static_cast<long>(b) * a.pitch + h), a.dt_bias[h], a.A_log[h]);
  for (int i = tid; i < 2 * D + ncol; i += 256) {
    if (i < D) {
      sk[i] = conv_one(a.B, kh * D + i, H * DV + kh * D + i, first);
    } else if (i < 2 * D) {
      sq[i - D] = conv_one(a.C, kh * D + i - D, H * DV + G * D + kh * D + i - D, first);
    } else {
      const int c = i - 2 * D;
      const float x = conv_one(a.x, h * DV + c0 + c, h * DV + c0 + c, true);
      sx[c] = x;
      su[c] = x * gate.y;
    }
  }
  __syncthreads();
  const float o = step_columns<VEC>(s.state + ((static_cast<long>(slot) * H + h) * D) * DV + c0, DV, ncol, D, s.lpr, pos > 0, gate.x, sq, sk, su, part);
  if (tid < ncol) out[tid] = fmaf(skip[h], sx[tid], o);
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
memory_step_kernel(const __grid_constant__ MemoryIn a, const __grid_constant__ Step s, float* __restrict__ norm, float* __restrict__ den) {
  __shared__ float sq[LS_MAX_D], sk[LS_MAX_D], su[LS_COLS], part[256 * VEC];
  const int b = blockIdx.x, h = blockIdx.y, H = a.H, D = a.D, DV = a.DV, tid = threadIdx.x;
  const bool is_n = static_cast<int>(blockIdx.z) == s.blocks;
  const int c0 = is_n ? 0 : blockIdx.z * LS_COLS, ncol = is_n ? 1 : min(LS_COLS, DV - c0);
  pdl_wait();
  pdl_launch_dependents();
  const int slot = s.slot[b];
  float* out = is_n ? den + static_cast<long>(b) * H + h : s.out + (static_cast<long>(b) * H + h) * DV + c0;
  if (!s.active[b] || slot < 0) {
    if (tid < ncol) out[tid] = is_n ? 1.f : 0.f;
    return;
  }
  const int pos = s.pos[b];
  const long row = static_cast<long>(b) * a.pitch, head = static_cast<long>(slot) * H + h;
  const float li = ls_cap(ls_load(reinterpret_cast<const T*>(a.i) + row + h) + a.i_b[h], a.cap);
  const float lf = ls_log_sigmoid(ls_cap(ls_load(reinterpret_cast<const T*>(a.f) + row + h) + a.f_b[h], a.cap));
  const float before = pos > 0 ? a.top[head * 2 + (pos & 1)] : 0.f, now = fmaxf(lf + before, li);
  const float f = expf(lf + before - now), w = expf(li - now), unit = 1.f / sqrtf(static_cast<float>(D));
  for (int i = tid; i < 2 * D + ncol; i += 256) {
    if (i < D) sk[i] = ls_load(reinterpret_cast<const T*>(a.k) + row + h * D + i);
    else if (i < 2 * D) sq[i - D] = ls_load(reinterpret_cast<const T*>(a.q) + row + h * D + i - D) * unit;
    else su[i - 2 * D] = is_n ? w : w * ls_load(reinterpret_cast<const T*>(a.v) + row + h * DV + c0 + i - 2 * D);
  }
  __syncthreads();
  if (is_n) {
    float o = 0.f;
    for (int r = tid; r < D; r += 256) {
      const float x = fmaf(pos > 0 ? norm[head * D + r] : 0.f, f, sk[r] * w);
      norm[head * D + r] = x;
      o = fmaf(x, sq[r], o);
    }
    o = block_sum<256>(o, part);
    if (tid == 0) {
      *out = fmaxf(fabsf(o), expf(-now)) + 1e-6f;
      a.top[head * 2 + ((pos + 1) & 1)] = now;
    }
    return;
  }
  const float o = step_columns<VEC>(s.state + head * D * DV + c0, DV, ncol, D, s.lpr, pos > 0, f, sq, sk, su, part);
  if (tid < ncol) out[tid] = o;
}

// ------------------------------------------------------------------------------------------------ norm and gate of parts of a row
// y = o (/ den); gate first: y = y act(z), then y / rms(y) * w; otherwise y / rms(y) * w * act(z). One warp per part of up to 512
// channels, else one CTA.
struct PartGate {
  const float *o, *den;  // [T, P, W], [T, P] or null
  const void *z, *w;     // [T, P W] rows z_pitch apart, [P W]
  void* out;             // [T, P W] rows out_pitch apart
  long parts, z_pitch, out_pitch;
  int P, W, sigmoid, gate_first;
  float eps, scale;
};

template <typename T>
__device__ __forceinline__ float part_act(float z, int sigmoid) {
  if constexpr (sizeof(T) == 2) return __fdividef(sigmoid ? 1.f : z, 1.f + __expf(-z));
  return sigmoid ? ls_sigmoid(z) : ls_silu(z);
}

template <typename T, int V, bool WARP>
__global__ void __launch_bounds__(256) part_gate_kernel(const __grid_constant__ PartGate a) {
  constexpr int LANES = WARP ? 32 : 256, KEEP = WARP ? 16 / V : 4;  // vectors a thread keeps between the two sweeps
  __shared__ float scratch[32];
  pdl_wait();
  pdl_launch_dependents();
  const long p = WARP ? static_cast<long>(blockIdx.x) * 8 + (threadIdx.x >> 5) : blockIdx.x;
  if (p >= a.parts) return;
  const int lane = WARP ? threadIdx.x & 31 : threadIdx.x, n = a.W / V;
  const long t = p / a.P;
  const int c0 = static_cast<int>(p - t * a.P) * a.W;
  const float* o = a.o + p * a.W;
  const T* z = reinterpret_cast<const T*>(a.z) + t * a.z_pitch + c0;
  const T* w = reinterpret_cast<const T*>(a.w) + c0;
  T* out = reinterpret_cast<T*>(a.out) + t * a.out_pitch + c0;
  const float div = a.den != nullptr ? 1.f / a.den[p] : 1.f;
  float keep[KEEP][V], gate[KEEP][V], ss = 0.f;
  auto load = [&](int c, float (&x)[V], float (&g)[V]) {
    ls_load_v<V>(o + c * V, x);
    ls_load_v<V>(z + c * V, g);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      g[i] = part_act<T>(g[i], a.sigmoid);
      x[i] *= a.gate_first ? div * g[i] : div;
    }
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = lane + j * LANES;
    if (c < n) {
      load(c, keep[j], gate[j]);
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(keep[j][i], keep[j][i], ss);
    }
  }
  for (int c = lane + KEEP * LANES; c < n; c += LANES) {
    float x[V], g[V];
    load(c, x, g);
#pragma unroll
    for (int i = 0; i < V; ++i) ss = fmaf(x[i], x[i], ss);
  }
  if constexpr (WARP) ss = warp_sum(ss);
  else ss = block_sum<256>(ss, scratch);
  const float r = a.scale / sqrtf(ss / a.W + a.eps);
  auto finish = [&](int c, float (&x)[V], float (&g)[V]) {
    float wt[V];
    ls_load_v<V>(w + c * V, wt);
#pragma unroll
    for (int i = 0; i < V; ++i) x[i] *= a.gate_first ? r * wt[i] : r * wt[i] * g[i];
    ls_store_v<V>(out + c * V, x);
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = lane + j * LANES;
    if (c < n) finish(c, keep[j], gate[j]);
  }
  for (int c = lane + KEEP * LANES; c < n; c += LANES) {
    float x[V], g[V];
    load(c, x, g);
    finish(c, x, g);
  }
}

template <typename... P>
static bool ls_aligned(int bytes, P... p) {
  return ((reinterpret_cast<uintptr_t>(p) | ... | uintptr_t(0)) % bytes) == 0;
}
static int ls_check(int H, int G, int D, int DV) { return H <= 0 || G <= 0 || H % G != 0 || D <= 0 || DV <= 0 || D > LS_MAX_D || H > 65535; }

template <typename T>
static int launch_ssd_prep(const SsdIn& a, const int* runs, const int* segs, int nruns, float* x, float* B, float* C, float4* gates, cudaStream_t s) {
  const int wx = a.H * a.DV, wb = a.G * a.D;
  const bool wide = wx % 4 == 0 && wb % 4 == 0 && a.pitch % 4 == 0 && ls_aligned(4 * sizeof(T), a.x, a.B, a.C, a.ring) && ls_aligned(16, x, B, C);
  const int V = wide ? 4 : 1;
  const dim3 grid(nruns, (wx + 2 * wb + 128 * V - 1) / (128 * V) + 1);
  auto kern = a.taps <= 4 ? (wide ? ssd_prep_kernel<T, 4, 4> : ssd_prep_kernel<T, 1, 4>) : (wide ? ssd_prep_kernel<T, 4, 0> : ssd_prep_kernel<T, 1, 0>);
  return (int)launch_pdl(kern, grid, dim3(128), 0, s, a, reinterpret_cast<const int4*>(runs), reinterpret_cast<const int4*>(segs), x, B, C, gates);
}

template <typename T>
static int launch_memory_prep(const MemoryIn& a, const int* segs, int nseg, int rows, float* q, float* k, float* v, float4* gates, cudaStream_t s) {
  const bool wide = a.D % 4 == 0 && a.DV % 4 == 0 && a.pitch % 4 == 0 && ls_aligned(4 * sizeof(T), a.q, a.k, a.v) && ls_aligned(16, q, k, v);
  const int gate_ctas = (nseg * a.H + 7) / 8;
  const long want = (static_cast<long>(rows) * a.H * (2 * a.D + a.DV) / (wide ? 4 : 1) + 255) / 256;
  const dim3 grid(gate_ctas + static_cast<unsigned>(want < 148 * 8 ? want : 148 * 8));
  auto kern = wide ? memory_prep_kernel<T, 4> : memory_prep_kernel<T, 1>;
  return (int)launch_pdl(kern, grid, dim3(256), 0, s, a, reinterpret_cast<const int4*>(segs), nseg, rows, gate_ctas, q, k, v, gates);
}

// WARPS: of a CTA with all its columns; narrow heads take fewer.
template <int RG, int NR, int CPT, int WARPS, int CTAS>
static int launch_linear_scan(Scan a, int nseg, cudaStream_t s) {
  constexpr int per = 32 / RG * CPT;  // columns of a warp
  int warps = WARPS;
  while (warps > 1 && warps / 2 * per >= a.DV) warps /= 2;
  const int cols = warps * per, bytes = LS_STAGES * LsSmem<RG, NR>::stage_floats(cols) * 4;
  auto kern = linear_scan_kernel<RG, NR, CPT, WARPS * 32, CTAS>;
  if (cudaError_t e = ensure_dynamic_smem(reinterpret_cast<const void*>(kern), LS_STAGES * LsSmem<RG, NR>::stage_floats(WARPS * per) * 4); e != cudaSuccess)
    return (int)e;
  a.blocks = (a.DV + cols - 1) / cols;
  // A plain launch: CTAs that start while the previous kernel still holds most of the machine would pile up on the few SMs
  // that are free, and stay there for the whole sequence.
  kern<<<dim3(a.blocks + (a.norm != nullptr ? 1 : 0), a.H, nseg), warps * 32, bytes, s>>>(a);
  return (int)cudaGetLastError();
}

// Columns of a step's CTA rows and lanes per row: VEC 4 where the widths allow it.
static int step_lanes(int DV, int vec) {
  const int c = DV < LS_COLS ? DV : LS_COLS;
  int l = 1;
  while (l * vec < c) l *= 2;
  return l;
}

template <typename T>
static int launch_part_gate(const PartGate& a, cudaStream_t s) {
  const bool wide = a.W % 4 == 0 && a.z_pitch % 4 == 0 && a.out_pitch % 4 == 0 && ls_aligned(4 * sizeof(T), a.z, a.w, a.out) && ls_aligned(16, a.o);
  if (a.W <= 512) {
    auto kern = wide ? part_gate_kernel<T, 4, true> : part_gate_kernel<T, 1, true>;
    return (int)launch_pdl(kern, dim3(static_cast<unsigned>((a.parts + 7) / 8)), dim3(256), 0, s, a);
  }
  auto kern = wide ? part_gate_kernel<T, 4, false> : part_gate_kernel<T, 1, false>;
  return (int)launch_pdl(kern, dim3(static_cast<unsigned>(a.parts)), dim3(256), 0, s, a);
}

}  // namespace sb

// runs: nruns x int4 (first row, tokens, first position, request); segs: one int4 per request (first row, tokens, first position, state
// slot). Outputs fp32: x [T, H DV], B and C [T, G D], gates [T, H] x 4. f32: element type of the projections, conv weights and ring.
extern "C" int sb_ssd_prep(const void* x, const void* B, const void* C, const void* dt, long pitch, const void* conv, const void* conv_b,
                           const float* A_log, const float* dt_bias, const void* ring, const int* runs, const int* segs, int nruns,
                           float* x_out, float* B_out, float* C_out, void* gates, int H, int G, int D, int DV, int taps, int f32,
                           cudaStream_t s) {
  if (nruns == 0) return 0;
  if (sb::ls_check(H, G, D, DV) || taps < 1 || taps > sb::LS_MAX_TAPS) return (int)cudaErrorInvalidValue;
  const sb::SsdIn a{x, B, C, dt, pitch, conv, conv_b, A_log, dt_bias, ring, H, G, D, DV, taps};
  if (f32) return sb::launch_ssd_prep<float>(a, runs, segs, nruns, x_out, B_out, C_out, (float4*)gates, s);
  return sb::launch_ssd_prep<__nv_bfloat16>(a, runs, segs, nruns, x_out, B_out, C_out, (float4*)gates, s);
}

extern "C" int sb_memory_prep(const void* q, const void* k, const void* v, const void* i, const void* f, long pitch, const float* i_b,
                              const float* f_b, float* top, const int* segs, int nseg, int rows, float* q_out, float* k_out, float* v_out,
                              void* gates, int H, int D, int DV, float cap, int f32, cudaStream_t s) {
  if (nseg == 0) return 0;
  if (sb::ls_check(H, H, D, DV) || !(cap > 0.f)) return (int)cudaErrorInvalidValue;
  const sb::MemoryIn a{q, k, v, i, f, pitch, i_b, f_b, top, H, D, DV, cap};
  if (f32) return sb::launch_memory_prep<float>(a, segs, nseg, rows, q_out, k_out, v_out, (float4*)gates, s);
  return sb::launch_memory_prep<__nv_bfloat16>(a, segs, nseg, rows, q_out, k_out, v_out, (float4*)gates, s);
}

// q, k [T, G D], v [T, H DV] fp32, gates [T, H] x 4 as the prep kernels wrote them; skip [H] or null; norm [slots, H, D] and den [T, H]
// or null; ring (null: none) with the projections in0 .. in2 of widths w0 .. w2 whose last rows it keeps.
extern "C" int sb_linear_scan(const float* q, const float* k, const float* v, const void* gates, const float* skip, float* out, float* state,
                              float* norm, float* den, const int* segs, int nseg, int H, int G, int D, int DV, void* ring, const void* in0,
                              const void* in1, const void* in2, long in_pitch, int w0, int w1, int w2, int taps, int esize, cudaStream_t s) {
  if (nseg == 0) return 0;
  if (sb::ls_check(H, G, D, DV) || nseg > 65535 || (norm != nullptr) != (den != nullptr) || !sb::ls_aligned(16, q, k, v, gates))
    return (int)cudaErrorInvalidValue;
  const sb::Scan a{q, k, v, (const float4*)gates, skip, out, state, norm, den, reinterpret_cast<const int4*>(segs), H, G, D, DV, 0,
                   ring, {in0, in1, in2}, in_pitch, {w0, w1, w2}, taps, esize};
  if (D <= 32) return sb::launch_linear_scan<8, 4, 4, 4, 4>(a, nseg, s);
  if (D <= 64) return sb::launch_linear_scan<16, 4, 8, 4, 4>(a, nseg, s);
  // a CTA of 64 columns has an SM to itself: more warps with fewer columns per lane hide more of a token's latency
  const bool few = static_cast<long>(nseg) * H * ((DV + 63) / 64 + (norm != nullptr ? 1 : 0)) <= 148;
  if (few && D <= 128) return sb::launch_linear_scan<16, 8, 4, 8, 1>(a, nseg, s);
  if (few && D <= 256) return sb::launch_linear_scan<16, 16, 4, 8, 1>(a, nseg, s);
  if (D <= 128) return sb::launch_linear_scan<16, 8, 8, 4, 4>(a, nseg, s);
  if (D <= 256) return sb::launch_linear_scan<32, 8, 8, 8, 2>(a, nseg, s);
  return sb::launch_linear_scan<32, 16, 4, 8, 1>(a, nseg, s);
}

// One token per row: slot / active / pos [B]; rows that are not active leave every state alone. out [B, H, DV] fp32.
extern "C" int sb_ssd_step(const void* x, const void* Bm, const void* C, const void* dt, long pitch, const void* conv, const void* conv_b,
                           const float* A_log, const float* dt_bias, const float* skip, void* ring, float* state, const int* slot,
                           const int* active, const int* pos, float* out, int B, int H, int G, int D, int DV, int taps, int f32,
                           cudaStream_t s) {
  if (B == 0) return 0;
  if (sb::ls_check(H, G, D, DV) || taps < 1 || taps > sb::LS_MAX_TAPS) return (int)cudaErrorInvalidValue;
  const sb::SsdIn a{x, Bm, C, dt, pitch, conv, conv_b, A_log, dt_bias, ring, H, G, D, DV, taps};
  const bool wide = DV % 4 == 0 && sb::ls_aligned(16, state);
  const int blocks = (DV + sb::LS_COLS - 1) / sb::LS_COLS;
  const sb::Step st{state, slot, active, pos, out, H, G, D, DV, blocks, sb::step_lanes(DV, wide ? 4 : 1)};
  const dim3 grid(B, H, blocks);
  using bf16 = __nv_bfloat16;
  auto kern = f32 ? (wide ? sb::ssd_step_kernel<float, 4> : sb::ssd_step_kernel<float, 1>)
                  : (wide ? sb::ssd_step_kernel<bf16, 4> : sb::ssd_step_kernel<bf16, 1>);
  return (int)sb::launch_pdl(kern, grid, dim3(256), 0, s, a, st, skip);
}

extern "C" int sb_memory_step(const void* q, const void* k, const void* v, const void* i, const void* f, long pitch, const float* i_b,
                              const float* f_b, float* top, float* state, float* norm, const int* slot, const int* active, const int* pos,
                              float* out, float* den, int B, int H, int D, int DV, float cap, int f32, cudaStream_t s) {
  if (B == 0) return 0;
  if (sb::ls_check(H, H, D, DV) || !(cap > 0.f)) return (int)cudaErrorInvalidValue;
  const sb::MemoryIn a{q, k, v, i, f, pitch, i_b, f_b, top, H, D, DV, cap};
  const bool wide = DV % 4 == 0 && sb::ls_aligned(16, state);
  const int blocks = (DV + sb::LS_COLS - 1) / sb::LS_COLS;
  const sb::Step st{state, slot, active, pos, out, H, H, D, DV, blocks, sb::step_lanes(DV, wide ? 4 : 1)};
  const dim3 grid(B, H, blocks + 1);
  using bf16 = __nv_bfloat16;
  auto kern = f32 ? (wide ? sb::memory_step_kernel<float, 4> : sb::memory_step_kernel<float, 1>)
                  : (wide ? sb::memory_step_kernel<bf16, 4> : sb::memory_step_kernel<bf16, 1>);
  return (int)sb::launch_pdl(kern, grid, dim3(256), 0, s, a, st, norm, den);
}

// o [T, P, W] fp32, den [T, P] or null, z [T, P W] and w [P W] of type T, out [T, P W].
extern "C" int sb_part_gate(const float* o, const float* den, const void* z, const void* w, void* out, int T, int P, int W, long z_pitch,
                            long out_pitch, float eps, float scale, int sigmoid, int gate_first, int f32, cudaStream_t s) {
  if (T == 0) return 0;
  if (P <= 0 || W <= 0) return (int)cudaErrorInvalidValue;
  const sb::PartGate a{o, den, z, w, out, static_cast<long>(T) * P, z_pitch, out_pitch, P, W, sigmoid, gate_first, eps, scale};
  return f32 ? sb::launch_part_gate<float>(a, s) : sb::launch_part_gate<__nv_bfloat16>(a, s);
}
