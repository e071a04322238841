// Kernels around an fp32 residual stream, for layers that normalise before and after every sub-layer:
//   * sb_stream_norm  one launch between two sub-layers: (mixture-of-experts combine, gated shared expert,) post-norm,
//                     residual add in fp32, pre-norm of the next sub-layer. With `ids` it gathers embedding rows instead
//                     and starts the stream; a second table can add a row chosen by (previous token, token).
//                     Norms treat a row as a whole or in equal parts; without a pre-norm the next sub-layer gets the stream itself.
//   * sb_glu          activation of a feed-forward, gated or not (silu, tanh-gelu, squared relu)
//   * sb_poly_norm    activation a N(z) + b N(z^2) + c N(z^3) + e of whole rows, N dividing by the root mean square
//   * sb_softcap      c tanh(x / c), in place
//   * sb_kv_scatter   new key / value rows into their cache slots, widths and element size free
//   * sb_heads        RMS norm (per head, or over all heads at once) and rotation of new queries and keys; keys and values into
//                     their cache slots; queries of differential attention spread over key pairs
//   * sb_latent_place norms of a token's query and key/value latents, rotation of its shared key part, cache write
//   * sb_latent_turn  rotation of the rotated part of latent queries, in place or beside absorbed queries
// Element types are bf16 or fp32 throughout (fp32: the engine's full-precision mode); all arithmetic is fp32.
#include "common.cuh"

namespace sb {

template <typename T>
__device__ __forceinline__ float to_f(T v);
template <>
__device__ __forceinline__ float to_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

template <typename T, int VEC>
__device__ __forceinline__ void load_vec(const T* p, float (&f)[VEC]) {
  if constexpr (VEC == 8 && sizeof(T) == 2) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y), c = unpack_bf16x2(u.z), d = unpack_bf16x2(u.w);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
  } else if constexpr (VEC == 8) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) f[i] = to_f(p[i]);
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void store_vec(T* p, const float (&f)[VEC]) {
  if constexpr (VEC == 8 && sizeof(T) == 2) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
  } else if constexpr (VEC == 8) {
    reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) p[i] = from_f<T>(f[i]);
  }
}

struct StreamNorm {
  const void* y;         // sub-layer output [T, H]; with `ids` an embedding table; with `dest` the experts' rows
  const int* ids;        // row of y per token (null: the token's own row); ids outside [0, y_rows) give a zero row
  const int* dest;       // [T, k] rows of y of a token's experts, < 0: none (null: no mixture of experts)
  const float* wts;      // [T, k] their weights
  const void* shared;    // [T, H] shared expert's output, same type as y, or null
  const float* gate;     // gate[t * gate_ld]: logit of the shared expert's gate, or null (gate 1)
  const void* post_w;    // norm of the sub-layer output, or null
  float* res;            // [T, H] residual stream, updated in place
  const void* pre_w;     // norm of the next sub-layer's input, or null
  void* h;               // [T, H] normed input of the next sub-layer (the stream itself without pre_w), or null
  int k, y_rows, gate_ld, init, layer_norm, H;  // init: the stream starts here (res is written, not added to)
  float eps, w_off;      // w_off is added to every norm weight
  const float* plus;     // [T, H] fp32 added to the sub-layer output (a mixer's, beside the experts), or null
  float h_scale;         // factor of h
  int groups;            // equal parts of a row with a norm of their own
  // second embedding table: row (prev * mul_prev + token * mul_cur) mod pair_rows is added to the sub-layer output, row
  // pair_rows where there is no previous token (prev < 0)
  const void* pair;      // same type as y, or null
  const int *pair_ids, *prev;
  long mul_prev, mul_cur;
  int pair_rows;
};

constexpr int STREAM_MAX_H = 8192;

// The same with an RMS norm of its own for each of `groups` parts: sums of squares by vector in shared memory, a warp per part. A vector
// lies in one part.
template <typename TW, int VEC, int MAXI, int THREADS>
__device__ __forceinline__ void row_norm_parts(float (&v)[MAXI][VEC], const TW* w, int H, int nvec, float eps, float w_off, int groups,
                                               float* part, float (&o)[MAXI][VEC]) {
  __syncthreads();  // an earlier use of `part`
#pragma unroll
  for (int j = 0; j < MAXI; ++j) {
    const int c = threadIdx.x + j * THREADS;
    if (c < nvec) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(v[j][i], v[j][i], ss);
      part[c] = ss;
    }
  }
  __syncthreads();
  const int per = nvec / groups, lane = threadIdx.x & 31;
  for (int g = threadIdx.x >> 5; g < groups; g += THREADS / 32) {
    float ss = 0.f;
    for (int c = lane; c < per; c += 32) ss += part[g * per + c];
    ss = warp_sum(ss);
    if (lane == 0) part[g * per] = 1.f / sqrtf(ss / (H / groups) + eps);
  }
  __syncthreads();
#pragma unroll
  for (int j = 0; j < MAXI; ++j) {
    const int c = threadIdx.x + j * THREADS;
    if (c < nvec) {
      const float rstd = part[c / per * per];
      float g[VEC];
      load_vec<TW, VEC>(w + static_cast<size_t>(c) * VEC, g);
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[j][i] = v[j][i] * rstd * (g[i] + w_off);
    }
  }
}

// v <- norm(v) * w over the row held by the CTA (thread t holds vectors t, t + THREADS, ...).
template <typename TW, int VEC, int MAXI, int THREADS>
__device__ __forceinline__ void row_norm(float (&v)[MAXI][VEC], const TW* w, int H, int nvec, float eps, float w_off, int layer_norm,
                                         float* scratch, float (&o)[MAXI][VEC]) {
  float mean = 0.f;
  if (layer_norm) {
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < MAXI; ++j)
      if (static_cast<int>(threadIdx.x) + j * THREADS < nvec)
#pragma unroll
        for (int i = 0; i < VEC; ++i) s += v[j][i];
    mean = block_sum<THREADS>(s, scratch) / H;
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < MAXI; ++j)
    if (static_cast<int>(threadIdx.x) + j * THREADS < nvec)
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const float d = v[j][i] - mean;
        ss += d * d;
      }
  const float rstd = 1.f / sqrtf(block_sum<THREADS>(ss, scratch) / H + eps);
#pragma unroll
  for (int j = 0; j < MAXI; ++j) {
    const int c = threadIdx.x + j * THREADS;
    if (c < nvec) {
      float g[VEC];
      load_vec<TW, VEC>(w + static_cast<size_t>(c) * VEC, g);
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[j][i] = (v[j][i] - mean) * rstd * (g[i] + w_off);
    }
  }
}

template <typename TY, typename TW, int VEC, int THREADS, bool PARTS>
__global__ void __launch_bounds__(THREADS) stream_norm_kernel(const __grid_constant__ StreamNorm a) {
  constexpr int MAXI = 32 / VEC;
  __shared__ float scratch[PARTS ? STREAM_MAX_H / VEC : 32];
  pdl_wait();  // inputs come from the previous kernel in the stream
  pdl_launch_dependents();
  const size_t row = blockIdx.x;
  const int H = a.H, nvec = H / VEC;
  const TY* y = reinterpret_cast<const TY*>(a.y);
  const TY* shared = reinterpret_cast<const TY*>(a.shared);
  size_t src = row;
  bool have = true;
  if (a.ids != nullptr) {
    const int id = a.ids[row];
    have = id >= 0 && id < a.y_rows;
    src = have ? id : 0;
  }
  const TY* pair = nullptr;
  if (a.pair != nullptr) {
    const int id = a.pair_ids[row], prev = a.prev[row];
    long r = a.pair_rows;
    if (prev >= 0) {
      r = (prev * a.mul_prev + id * a.mul_cur) % a.pair_rows;
      if (r < 0) r += a.pair_rows;
    }
    pair = reinterpret_cast<const TY*>(a.pair) + r * H;
  }
  const float gate = (shared != nullptr && a.gate != nullptr) ? 1.f / (1.f + expf(-a.gate[row * a.gate_ld])) : 1.f;
  float v[MAXI][VEC];
#pragma unroll
  for (int j = 0; j < MAXI; ++j) {
    const int c = threadIdx.x + j * THREADS;
    if (c < nvec) {
      const size_t off = static_cast<size_t>(c) * VEC;
      if (a.dest != nullptr) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[j][i] = 0.f;
        for (int r = 0; r < a.k; ++r) {  // route order: the same sum whatever the batch
          const int d = a.dest[row * a.k + r];
          if (d < 0) continue;
          const float wt = a.wts[row * a.k + r];
          float e[VEC];
          load_vec<TY, VEC>(y + static_cast<size_t>(d) * H + off, e);
#pragma unroll
          for (int i = 0; i < VEC; ++i) v[j][i] = fmaf(wt, e[i], v[j][i]);
        }
        if (shared != nullptr) {
          float e[VEC];
          load_vec<TY, VEC>(shared + row * H + off, e);
#pragma unroll
          for (int i = 0; i < VEC; ++i) v[j][i] = fmaf(gate, e[i], v[j][i]);
        }
      } else if (have) {
        load_vec<TY, VEC>(y + src * H + off, v[j]);
      } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[j][i] = 0.f;
      }
      if (a.plus != nullptr) {
        float e[VEC];
        load_vec<float, VEC>(a.plus + row * H + off, e);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[j][i] += e[i];
      }
      if (pair != nullptr) {
        float e[VEC];
        load_vec<TY, VEC>(pair + off, e);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[j][i] += e[i];
      }
    }
  }
  if (a.post_w != nullptr) {
    if constexpr (PARTS) row_norm_parts<TW, VEC, MAXI, THREADS>(v, reinterpret_cast<const TW*>(a.post_w), H, nvec, a.eps, a.w_off, a.groups, scratch, v);
    else row_norm<TW, VEC, MAXI, THREADS>(v, reinterpret_cast<const TW*>(a.post_w), H, nvec, a.eps, a.w_off, a.layer_norm, scratch, v);
  }
#pragma unroll
  for (int j = 0; j < MAXI; ++j) {
    const int c = threadIdx.x + j * THREADS;
    if (c < nvec) {
      float* rp = a.res + row * H + static_cast<size_t>(c) * VEC;
      if (!a.init) {
        float r[VEC];
        load_vec<float, VEC>(rp, r);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[j][i] += r[i];
      }
      store_vec<float, VEC>(rp, v[j]);
    }
  }
  if (a.h != nullptr) {
    float o[MAXI][VEC];
    if (a.pre_w == nullptr) {
#pragma unroll
      for (int j = 0; j < MAXI; ++j)
#pragma unroll
        for (int i = 0; i < VEC; ++i) o[j][i] = v[j][i];
    } else if constexpr (PARTS) {
      row_norm_parts<TW, VEC, MAXI, THREADS>(v, reinterpret_cast<const TW*>(a.pre_w), H, nvec, a.eps, a.w_off, a.groups, scratch, o);
    } else {
      row_norm<TW, VEC, MAXI, THREADS>(v, reinterpret_cast<const TW*>(a.pre_w), H, nvec, a.eps, a.w_off, a.layer_norm, scratch, o);
    }
    TW* h = reinterpret_cast<TW*>(a.h);
#pragma unroll
    for (int j = 0; j < MAXI; ++j) {
      const int c = threadIdx.x + j * THREADS;
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[j][i] *= a.h_scale;
      if (c < nvec) store_vec<TW, VEC>(h + row * H + static_cast<size_t>(c) * VEC, o[j]);
    }
  }
}

template <typename TY, typename TW, bool PARTS>
static int launch_stream_norm_form(const StreamNorm& a, int T, bool vec, cudaStream_t s) {
  if (vec && a.H <= 1024)
    return (int)launch_pdl(stream_norm_kernel<TY, TW, 8, 128, PARTS>, dim3(T), dim3(128), 0, s, a);
  if (vec) return (int)launch_pdl(stream_norm_kernel<TY, TW, 8, 256, PARTS>, dim3(T), dim3(256), 0, s, a);
  return (int)launch_pdl(stream_norm_kernel<TY, TW, 1, 256, PARTS>, dim3(T), dim3(256), 0, s, a);
}
template <typename TY, typename TW>
static int launch_stream_norm(const StreamNorm& a, int T, bool vec, cudaStream_t s) {
  if (a.groups > 1) return launch_stream_norm_form<TY, TW, true>(a, T, vec && a.H / a.groups % 8 == 0, s);
  return launch_stream_norm_form<TY, TW, false>(a, T, vec, s);
}

enum : int { ACT_SILU = 0, ACT_GELU_TANH = 1, ACT_RELU2 = 2 };

__device__ __forceinline__ float activate(float z, int act) {
  if (act == ACT_SILU) return z / (1.f + expf(-z));
  if (act == ACT_GELU_TANH) return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
  const float r = fmaxf(z, 0.f);
  return r * r;
}

// out[t, f] = act(in[t, f]) * up[t, f], or act(in[t, f]) where up is null; rows of in and up are in_pitch apart
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
glu_kernel(const T* __restrict__ in, const T* __restrict__ up, T* __restrict__ out, long rows, int F, long in_pitch, long out_pitch, int act) {
  pdl_wait();
  pdl_launch_dependents();
  const int nv = F / VEC;
  const long n = rows * nv;
  for (long i = static_cast<long>(blockIdx.x) * 256 + threadIdx.x; i < n; i += static_cast<long>(gridDim.x) * 256) {
    const long t = i / nv;
    const int c = static_cast<int>(i - t * nv) * VEC;
    float g[VEC];
    load_vec<T, VEC>(in + t * in_pitch + c, g);
#pragma unroll
    for (int j = 0; j < VEC; ++j) g[j] = activate(g[j], act);
    if (up != nullptr) {
      float u[VEC];
      load_vec<T, VEC>(up + t * in_pitch + c, u);
#pragma unroll
      for (int j = 0; j < VEC; ++j) g[j] *= u[j];
    }
    store_vec<T, VEC>(out + t * out_pitch + c, g);
  }
}

// Rows of F hidden units: a N(z) + b N(z^2) + c N(z^3) + e with N(x) = x / sqrt(mean(x^2) + eps) and (a, b, c, e) = coef. One CTA per row;
// the second sweep finds the row in the caches. sums: [T, 3] sums of z^2, z^4, z^6 over the whole row of `all` units (tensor-parallel
// ranks hold parts of it); null: computed here.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
poly_norm_kernel(const T* __restrict__ in, T* __restrict__ out, const float* __restrict__ coef, const float* __restrict__ sums, int F, int all,
                 long in_pitch, long out_pitch, float eps) {
  constexpr int KEEP = VEC == 8 ? 4 : 8;  // vectors a thread keeps between the sweeps
  __shared__ float scratch[32];
  pdl_wait();
  pdl_launch_dependents();
  const long t = blockIdx.x;
  const T* x = in + t * in_pitch;
  T* y = out + t * out_pitch;
  const int n = F / VEC;
  float keep[KEEP][VEC], s2 = 0.f, s4 = 0.f, s6 = 0.f;
  auto add = [&](const float (&z)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const float p2 = z[i] * z[i], p4 = p2 * p2;
      s2 += p2;
      s4 += p4;
      s6 = fmaf(p4, p2, s6);
    }
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = threadIdx.x + j * 256;
    if (c < n) {
      load_vec<T, VEC>(x + static_cast<long>(c) * VEC, keep[j]);
      if (sums == nullptr) add(keep[j]);
    }
  }
  if (sums == nullptr) {
    for (int c = threadIdx.x + KEEP * 256; c < n; c += 256) {
      float z[VEC];
      load_vec<T, VEC>(x + static_cast<long>(c) * VEC, z);
      add(z);
    }
    s2 = block_sum<256>(s2, scratch);
    s4 = block_sum<256>(s4, scratch);
    s6 = block_sum<256>(s6, scratch);
  } else {
    s2 = sums[3 * t];
    s4 = sums[3 * t + 1];
    s6 = sums[3 * t + 2];
  }
  const float a = coef[0] / sqrtf(s2 / all + eps), b = coef[1] / sqrtf(s4 / all + eps), c3 = coef[2] / sqrtf(s6 / all + eps), e = coef[3];
  auto put = [&](int c, float (&z)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) z[i] = fmaf(z[i], fmaf(z[i], fmaf(z[i], c3, b), a), e);
    store_vec<T, VEC>(y + static_cast<long>(c) * VEC, z);
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = threadIdx.x + j * 256;
    if (c < n) put(c, keep[j]);
  }
  for (int c = threadIdx.x + KEEP * 256; c < n; c += 256) {
    float z[VEC];
    load_vec<T, VEC>(x + static_cast<long>(c) * VEC, z);
    put(c, z);
  }
}

// x <- cap tanh(x / cap) over a row of n floats per y-block, rows `pitch` apart
__global__ void __launch_bounds__(256) softcap_kernel(float* __restrict__ x, long n, long pitch, float cap) {
  pdl_wait();
  pdl_launch_dependents();
  float* row = x + static_cast<long>(blockIdx.y) * pitch;
  const float inv = 1.f / cap;
  const bool vec = ((reinterpret_cast<uintptr_t>(row) & 15) | (n & 3)) == 0;
  const long step = static_cast<long>(gridDim.x) * 256, first = static_cast<long>(blockIdx.x) * 256 + threadIdx.x;
  for (long i = first; vec && i < n / 4; i += step) {
    float4 v = reinterpret_cast<float4*>(row)[i];
    v.x = cap * tanhf(v.x * inv);
    v.y = cap * tanhf(v.y * inv);
    v.z = cap * tanhf(v.z * inv);
    v.w = cap * tanhf(v.w * inv);
    reinterpret_cast<float4*>(row)[i] = v;
  }
  for (long i = first; !vec && i < n; i += step) row[i] = cap * tanhf(row[i] * inv);
}

// One CTA per token: `kb` bytes of its key row and `vb` bytes of its value row to cache slot slots[t] (< 0: skipped).
template <typename U>
__global__ void __launch_bounds__(128)
kv_scatter_kernel(const char* __restrict__ k, const char* __restrict__ v, const int* __restrict__ slots, char* __restrict__ k_cache,
                  char* __restrict__ v_cache, int kb, int vb, long k_pitch, long v_pitch) {
  pdl_wait();
  pdl_launch_dependents();
  const int slot = slots[blockIdx.x];
  if (slot < 0) return;
  const U* ks = reinterpret_cast<const U*>(k + blockIdx.x * k_pitch);
  const U* vs = reinterpret_cast<const U*>(v + blockIdx.x * v_pitch);
  U* kd = reinterpret_cast<U*>(k_cache + static_cast<long>(slot) * kb);
  U* vd = reinterpret_cast<U*>(v_cache + static_cast<long>(slot) * vb);
  const int nk = kb / sizeof(U), nv = vb / sizeof(U);
  for (int c = threadIdx.x; c < nk + nv; c += blockDim.x) {
    if (c < nk) kd[c] = ks[c];
    else vd[c - nk] = vs[c - nk];
  }
}

// New queries, keys and values of one attention layer. One warp per (token, head): query heads first, then key heads, then value
// heads. Query and key heads: RMS norm over D times q_norm / k_norm (null: none), then the first `dims` coordinates turned by
// the position's angles (table [positions, dims] = cos | sin of the dims / 2 pairs; pair i is (2i, 2i + 1) when interleaved,
// else (i, i + dims / 2)). Queries go to q_out (which may be q), keys and values to cache slot slots[t] (< 0: nowhere).
// maps = 2: query heads 2 i and 2 i + 1 meet the first and the second D coordinates of a key of 2 D: head h is written as a row of
// 2 D, zero in the other half; key heads 2 g and 2 g + 1 are the halves of one key. Hkv = Hv = 0: queries only.
struct Heads {
  const void *q, *k, *v;
  void* q_out;
  const void *q_norm, *k_norm;
  const float* table;
  const int *positions, *slots;
  void *k_cache, *v_cache;
  int Hq, Hkv, Hv, D, DV, dims, interleaved, maps;
  long q_pitch, k_pitch, v_pitch, q_out_pitch;
  float eps;
};
constexpr int HEADS_MAX_D = 512;

template <typename T>
__global__ void __launch_bounds__(128) heads_kernel(const __grid_constant__ Heads a) {
  __shared__ float x_s[4][HEADS_MAX_D];
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, vec = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (vec >= a.Hq + a.Hkv + a.Hv) return;
  const long t = blockIdx.x;
  const int slot = a.slots[t];
  if (vec >= a.Hq + a.Hkv) {
    const int h = vec - a.Hq - a.Hkv;
    if (slot < 0) return;
    const T* src = reinterpret_cast<const T*>(a.v) + t * a.v_pitch + static_cast<long>(h) * a.DV;
    T* dst = reinterpret_cast<T*>(a.v_cache) + (static_cast<long>(slot) * a.Hv + h) * a.DV;
    for (int d = lane; d < a.DV; d += 32) dst[d] = src[d];
    return;
  }
  const bool is_q = vec < a.Hq;
  const int h = is_q ? vec : vec - a.Hq;
  const T* src = is_q ? reinterpret_cast<const T*>(a.q) + t * a.q_pitch : reinterpret_cast<const T*>(a.k) + t * a.k_pitch;
  src += static_cast<long>(h) * a.D;
  const T* w = reinterpret_cast<const T*>(is_q ? a.q_norm : a.k_norm);
  float* x = x_s[threadIdx.x >> 5];
  float ss = 0.f;
  for (int d = lane; d < a.D; d += 32) {
    x[d] = to_f(src[d]);
    ss = fmaf(x[d], x[d], ss);
  }
  if (w != nullptr) {
    const float r = 1.f / sqrtf(warp_sum(ss) / a.D + a.eps);
    for (int d = lane; d < a.D; d += 32) x[d] *= r * to_f(w[d]);
  }
  __syncwarp();
  T* dst = is_q ? reinterpret_cast<T*>(a.q_out) + t * a.q_out_pitch + static_cast<long>(h) * a.maps * a.D
                : reinterpret_cast<T*>(a.k_cache) + (static_cast<long>(slot < 0 ? 0 : slot) * a.Hkv + h) * a.D;
  if (!is_q && slot < 0) return;
  if (is_q && a.maps == 2) {
    T* zero = h & 1 ? dst : dst + a.D;
    dst += h & 1 ? a.D : 0;
    for (int d = lane; d < a.D; d += 32) zero[d] = from_f<T>(0.f);
  }
  const int half = a.dims / 2;
  const float* cs = half > 0 ? a.table + static_cast<long>(a.positions[t]) * a.dims : nullptr;
  for (int d = lane; d < a.D; d += 32) {
    float y = x[d];
    if (d < a.dims) {
      const int i = a.interleaved ? d >> 1 : (d < half ? d : d - half);
      const bool second = a.interleaved ? d & 1 : d >= half;
      const float other = x[a.interleaved ? d ^ 1 : (second ? d - half : d + half)];
      y = second ? fmaf(other, cs[half + i], y * cs[i]) : fmaf(-other, cs[half + i], y * cs[i]);
    }
    dst[d] = from_f<T>(y);
  }
}

// The same for the usual widths, 8 elements per lane and 32 / L heads per warp: L = D / 8 lanes have a query or key head (L a power
// of two; halves of a rotation are whole vectors), the value heads follow as one row of Hv * DV elements.
template <typename T, int L>
__global__ void __launch_bounds__(256) heads_wide_kernel(const __grid_constant__ Heads a) {
  constexpr int D = 8 * L;
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x % L;
  const long t = blockIdx.x;
  const int slot = a.slots[t], heads = a.Hq + a.Hkv, half = a.dims / 2, c0 = lane * 8;
  const float* cs = half > 0 ? a.table + static_cast<long>(a.positions[t]) * a.dims : nullptr;
  // a lane's part of the rotation is the same for every head: pair of element i, and whether it is the second of its pair
  float cosv[8], sinv[8];
  const bool turned = c0 < a.dims;
  const int away = a.interleaved || !turned ? 0 : half / 8;  // lanes to the other half
  const bool second = turned && !a.interleaved && c0 >= half;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int p = a.interleaved ? (c0 + i) / 2 : second ? c0 + i - half : c0 + i;
    cosv[i] = turned ? cs[p] : 1.f;
    sinv[i] = turned ? cs[half + p] : 0.f;
    if (a.interleaved ? !(i & 1) : !second) sinv[i] = -sinv[i];
  }
  const int rounds = (heads * L + 255) / 256;  // whole warps stay together for the exchanges
  for (int r = 0; r < rounds; ++r) {
    const int vec = (r * 256 + static_cast<int>(threadIdx.x)) / L;
    const bool on = vec < heads, is_q = vec < a.Hq;
    const int h = is_q ? vec : vec - a.Hq;
    float x[8], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) x[i] = 0.f;
    if (on) load_vec<T, 8>((is_q ? reinterpret_cast<const T*>(a.q) + t * a.q_pitch : reinterpret_cast<const T*>(a.k) + t * a.k_pitch) + h * D + c0, x);
    const T* w = reinterpret_cast<const T*>(is_q ? a.q_norm : a.k_norm);
    if (a.q_norm != nullptr) {
#pragma unroll
      for (int i = 0; i < 8; ++i) ss = fmaf(x[i], x[i], ss);
#pragma unroll
      for (int o = 1; o < L; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (on && w != nullptr) {
        const float rs = 1.f / sqrtf(ss / D + a.eps);
        float g[8];
        load_vec<T, 8>(w + c0, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] *= rs * g[i];
      }
    }
    if (half > 0) {
      float other[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) other[i] = x[i ^ 1];
      if (!a.interleaved) {
        const int from = (threadIdx.x & 31) + (second ? -away : away);
#pragma unroll
        for (int i = 0; i < 8; ++i) other[i] = __shfl_sync(0xffffffffu, x[i], from & 31);
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) x[i] = fmaf(other[i], sinv[i], x[i] * cosv[i]);
    }
    if (!on || (!is_q && slot < 0)) continue;
    if (is_q) {
      T* dst = reinterpret_cast<T*>(a.q_out) + t * a.q_out_pitch + static_cast<long>(h) * a.maps * D + c0;
      if (a.maps == 2) {
        const float zero[8] = {};
        store_vec<T, 8>(h & 1 ? dst : dst + D, zero);
        dst += h & 1 ? D : 0;
      }
      store_vec<T, 8>(dst, x);
    } else {
      store_vec<T, 8>(reinterpret_cast<T*>(a.k_cache) + (static_cast<long>(slot) * a.Hkv + h) * D + c0, x);
    }
  }
  if (slot < 0) return;
  const int nv = a.Hv * a.DV;
  const T* v = reinterpret_cast<const T*>(a.v) + t * a.v_pitch;
  T* v_out = reinterpret_cast<T*>(a.v_cache) + static_cast<long>(slot) * nv;
  for (int c = threadIdx.x * 8; c < nv; c += 256 * 8) {
    float e[8];
    load_vec<T, 8>(v + c, e);
    store_vec<T, 8>(v_out + c, e);
  }
}

template <typename T>
static int launch_heads(const Heads& a, int rows, cudaStream_t s) {
  const int L = a.D / 8, half = a.dims / 2;
  bool wide = a.D % 8 == 0 && (L == 4 || L == 8 || L == 16 || L == 32) && (a.Hv * a.DV) % 8 == 0 && a.q_pitch % 8 == 0 && a.k_pitch % 8 == 0 &&
              a.v_pitch % 8 == 0 && a.q_out_pitch % 8 == 0 && (a.interleaved ? a.dims : half) % 8 == 0;
  for (const void* x : {a.q, a.k, a.v, static_cast<const void*>(a.q_out), a.q_norm, a.k_norm, static_cast<const void*>(a.k_cache), static_cast<const void*>(a.v_cache)})
    wide = wide && (reinterpret_cast<uintptr_t>(x) & 15) == 0;
  if (!wide) return (int)launch_pdl(heads_kernel<T>, dim3(rows, (a.Hq + a.Hkv + a.Hv + 3) / 4), dim3(128), 0, s, a);
  auto kern = L == 4 ? heads_wide_kernel<T, 4> : L == 8 ? heads_wide_kernel<T, 8> : L == 16 ? heads_wide_kernel<T, 16> : heads_wide_kernel<T, 32>;
  return (int)launch_pdl(kern, dim3(rows), dim3(256), 0, s, a);
}

// The same with one norm over all query heads and one over all key heads (a weight per channel): one CTA per token, its rows
// staged in shared memory as they came. sums: [T, 2] sums of squares of the whole projections (tensor-parallel ranks hold
// parts of them) with q_all / k_all channels; null: computed here.
struct HeadsAll {
  Heads h;
  const float* sums;
  int q_all, k_all;
};
constexpr int HEADS_ALL_THREADS = 256;

template <typename T, int VEC>
__global__ void __launch_bounds__(HEADS_ALL_THREADS) heads_all_kernel(const __grid_constant__ HeadsAll p) {
  const Heads& a = p.h;
  extern __shared__ __align__(16) unsigned char raw_s[];
  T* x = reinterpret_cast<T*>(raw_s);
  __shared__ float scratch[32];
  pdl_wait();
  pdl_launch_dependents();
  const long t = blockIdx.x;
  const int nq = a.Hq * a.D, nk = a.Hkv * a.D, nv = a.Hkv * a.DV;
  const T* q = reinterpret_cast<const T*>(a.q) + t * a.q_pitch;
  const T* k = reinterpret_cast<const T*>(a.k) + t * a.k_pitch;
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * VEC; c < nq + nk; c += HEADS_ALL_THREADS * VEC) {
    float e[VEC];
    load_vec<T, VEC>(c < nq ? q + c : k + (c - nq), e);
    store_vec<T, VEC>(x + c, e);
#pragma unroll
    for (int i = 0; i < VEC; ++i) (c < nq ? sq : sk) += e[i] * e[i];
  }
  if (p.sums != nullptr) {
    sq = p.sums[2 * t];
    sk = p.sums[2 * t + 1];
    __syncthreads();
  } else {
    sq = block_sum<HEADS_ALL_THREADS>(sq, scratch);
    sk = block_sum<HEADS_ALL_THREADS>(sk, scratch);
  }
  const float rq = 1.f / sqrtf(sq / p.q_all + a.eps), rk = 1.f / sqrtf(sk / p.k_all + a.eps);
  const int slot = a.slots[t];
  const int half = a.dims / 2;
  const float* cs = half > 0 ? a.table + static_cast<long>(a.positions[t]) * a.dims : nullptr;
  T* q_out = reinterpret_cast<T*>(a.q_out) + t * a.q_pitch;
  T* k_out = reinterpret_cast<T*>(a.k_cache) + static_cast<long>(slot < 0 ? 0 : slot) * nk;
  for (int c = threadIdx.x * VEC; c < nq + nk; c += HEADS_ALL_THREADS * VEC) {
    const bool is_q = c < nq;
    if (!is_q && slot < 0) break;
    const T* w = reinterpret_cast<const T*>(is_q ? a.q_norm : a.k_norm) + (is_q ? c : c - nq);
    const float r = is_q ? rq : rk;
    float y[VEC], g[VEC];
    load_vec<T, VEC>(x + c, y);
    load_vec<T, VEC>(w, g);
    const int d0 = (is_q ? c : c - nq) % a.D;  // VEC divides D: a vector lies in one head
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      y[i] *= r * g[i];
      const int d = d0 + i;
      if (d < a.dims) {
        const int pair = a.interleaved ? d >> 1 : (d < half ? d : d - half);
        const bool second = a.interleaved ? d & 1 : d >= half;
        const int away = a.interleaved ? (d ^ 1) - d : (second ? -half : half);
        const float other = to_f(x[c + i + away]) * r * to_f(w[i + away]);
        y[i] = second ? fmaf(other, cs[half + pair], y[i] * cs[pair]) : fmaf(-other, cs[half + pair], y[i] * cs[pair]);
      }
    }
    store_vec<T, VEC>(is_q ? q_out + c : k_out + (c - nq), y);
  }
  if (slot < 0) return;
  const T* v = reinterpret_cast<const T*>(a.v) + t * a.v_pitch;
  T* v_out = reinterpret_cast<T*>(a.v_cache) + static_cast<long>(slot) * nv;
  for (int c = threadIdx.x * VEC; c < nv; c += HEADS_ALL_THREADS * VEC) {
    float e[VEC];
    load_vec<T, VEC>(v + c, e);
    store_vec<T, VEC>(v_out + c, e);
  }
}

template <typename T>
static int launch_heads_all(const HeadsAll& p, int T_, bool vec, cudaStream_t s) {
  const int bytes = (p.h.Hq + p.h.Hkv) * p.h.D * static_cast<int>(sizeof(T));
  auto kern = vec ? heads_all_kernel<T, 8> : heads_all_kernel<T, 1>;
  if (bytes > 200 * 1024) return (int)cudaErrorInvalidValue;
  if (bytes > 40 * 1024)
    if (cudaError_t e = ensure_dynamic_smem(reinterpret_cast<const void*>(kern), 200 * 1024); e != cudaSuccess) return (int)e;
  return (int)launch_pdl(kern, dim3(T_), dim3(HEADS_ALL_THREADS), bytes, s, p);
}

// Latent attention, one CTA per token: the query latent dq [T, R1] is RMS normed into q_out; of dkv [T, R2 + dims] the first R2
// are RMS normed and the last `dims` turned, both into cache row slots[t] (< 0: nowhere) of width R2 + dims.
struct LatentPlace {
  const void *dq, *dkv, *q_norm, *kv_norm;
  const float* table;
  const int *positions, *slots;
  void *q_out, *cache;
  int R1, R2, dims, interleaved;
  long dq_pitch, dkv_pitch;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(128) latent_place_kernel(const __grid_constant__ LatentPlace a) {
  __shared__ float scratch[32];
  pdl_wait();
  pdl_launch_dependents();
  const long t = blockIdx.x;
  const int slot = a.slots[t];
  const float* cs = a.table + static_cast<long>(a.positions[t]) * a.dims;
  const T* dq = reinterpret_cast<const T*>(a.dq) + t * a.dq_pitch;
  const T* dkv = reinterpret_cast<const T*>(a.dkv) + t * a.dkv_pitch;
  float sq = 0.f, sk = 0.f;
#pragma unroll 4
  for (int c = threadIdx.x; c < a.R1; c += 128) {
    const float e = to_f(dq[c]);
    sq = fmaf(e, e, sq);
  }
#pragma unroll 4
  for (int c = threadIdx.x; c < a.R2; c += 128) {
    const float e = to_f(dkv[c]);
    sk = fmaf(e, e, sk);
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) {
    scratch[threadIdx.x >> 5] = sq;
    scratch[4 + (threadIdx.x >> 5)] = sk;
  }
  __syncthreads();
  const float rq = 1.f / sqrtf((scratch[0] + scratch[1] + scratch[2] + scratch[3]) / a.R1 + a.eps);
  const float rk = 1.f / sqrtf((scratch[4] + scratch[5] + scratch[6] + scratch[7]) / a.R2 + a.eps);
  const T* wq = reinterpret_cast<const T*>(a.q_norm);
  T* q_out = reinterpret_cast<T*>(a.q_out) + t * a.R1;
#pragma unroll 4
  for (int c = threadIdx.x; c < a.R1; c += 128) q_out[c] = from_f<T>(to_f(dq[c]) * rq * to_f(wq[c]));
  if (slot < 0) return;
  const T* wk = reinterpret_cast<const T*>(a.kv_norm);
  T* out = reinterpret_cast<T*>(a.cache) + static_cast<long>(slot) * (a.R2 + a.dims);
  const int half = a.dims / 2;
#pragma unroll 4
  for (int c = threadIdx.x; c < a.R2 + half; c += 128) {
    if (c < a.R2) {
      out[c] = from_f<T>(to_f(dkv[c]) * rk * to_f(wk[c]));
      continue;
    }
    const int i = c - a.R2, d0 = a.R2 + (a.interleaved ? 2 * i : i), d1 = a.R2 + (a.interleaved ? 2 * i + 1 : i + half);
    const float u = to_f(dkv[d0]), v = to_f(dkv[d1]), cosv = cs[i], sinv = cs[half + i];
    out[d0] = from_f<T>(u * cosv - v * sinv);
    out[d1] = from_f<T>(v * cosv + u * sinv);
  }
}

// Rotated part of latent queries: the last `dims` coordinates of every head of q [T, H, D + dims] are turned and written to the
// first `dims` coordinates behind dst [T, H, ...] (which may be the queries themselves). One thread per pair.
template <typename T>
__global__ void __launch_bounds__(256)
latent_turn_kernel(const T* __restrict__ q, T* __restrict__ dst, const float* __restrict__ table, const int* __restrict__ positions,
                   long pairs, int H, int D, int dims, int interleaved, long q_pitch, long q_head, long dst_pitch, long dst_head) {
  pdl_wait();
  pdl_launch_dependents();
  const int half = dims / 2;
  for (long n = static_cast<long>(blockIdx.x) * 256 + threadIdx.x; n < pairs; n += static_cast<long>(gridDim.x) * 256) {
    const int i = static_cast<int>(n % half);
    const long th = n / half;
    const int h = static_cast<int>(th % H);
    const long t = th / H;
    const float* cs = table + static_cast<long>(positions[t]) * dims;
    const int d0 = interleaved ? 2 * i : i, d1 = interleaved ? 2 * i + 1 : i + half;
    const T* src = q + t * q_pitch + h * q_head + D;
    T* out = dst + t * dst_pitch + h * dst_head;
    const float u = to_f(src[d0]), v = to_f(src[d1]);
    out[d0] = from_f<T>(u * cs[i] - v * cs[half + i]);
    out[d1] = from_f<T>(v * cs[i] + u * cs[half + i]);
  }
}

}  // namespace sb

// q_out (row pitch q_out_pitch): where the queries go; maps 1, or 2 for pairs (see Heads).
extern "C" int sb_heads(const void* q, const void* k, const void* v, void* q_out, const void* q_norm, const void* k_norm, const float* table,
                        const int* positions, const int* slots, void* k_cache, void* v_cache, int T, int Hq, int Hkv, int Hv, int D, int DV,
                        int dims, int interleaved, int maps, long q_pitch, long k_pitch, long v_pitch, long q_out_pitch, float eps, int f32,
                        cudaStream_t s) {
  if (T == 0) return 0;
  if (D <= 0 || D > sb::HEADS_MAX_D || DV <= 0 || dims < 0 || dims > D || dims % 2 || Hq <= 0 || Hkv < 0 || Hv < 0 || (maps != 1 && maps != 2) ||
      (maps == 2 && (Hq % 2 || q == q_out)))
    return (int)cudaErrorInvalidValue;
  const sb::Heads a{q, k, v, q_out, q_norm, k_norm, table, positions, slots, k_cache, v_cache, Hq, Hkv, Hv, D, DV, dims, interleaved, maps,
                    q_pitch, k_pitch, v_pitch, q_out_pitch, eps};
  return f32 ? sb::launch_heads<float>(a, T, s) : sb::launch_heads<__nv_bfloat16>(a, T, s);
}

// As sb_heads, with norms over all query heads and over all key heads (see HeadsAll).
extern "C" int sb_heads_all(void* q, const void* k, const void* v, const void* q_norm, const void* k_norm, const float* table,
                            const int* positions, const int* slots, void* k_cache, void* v_cache, int T, int Hq, int Hkv, int D, int DV,
                            int dims, int interleaved, long q_pitch, long k_pitch, long v_pitch, const float* sums, int q_all, int k_all,
                            float eps, int f32, cudaStream_t s) {
  if (T == 0) return 0;
  if (D <= 0 || DV <= 0 || dims < 0 || dims > D || dims % 2 || Hq <= 0 || Hkv <= 0 || q_norm == nullptr || k_norm == nullptr)
    return (int)cudaErrorInvalidValue;
  const sb::HeadsAll p{{q, k, v, q, q_norm, k_norm, table, positions, slots, k_cache, v_cache, Hq, Hkv, Hkv, D, DV, dims, interleaved, 1, q_pitch,
                        k_pitch, v_pitch, q_pitch, eps}, sums, q_all, k_all};
  bool vec = D % 8 == 0 && DV % 8 == 0 && q_pitch % 8 == 0 && k_pitch % 8 == 0 && v_pitch % 8 == 0;
  for (const void* x : {static_cast<const void*>(q), k, v, q_norm, k_norm, static_cast<const void*>(k_cache), static_cast<const void*>(v_cache)})
    vec = vec && (reinterpret_cast<uintptr_t>(x) & 15) == 0;
  return f32 ? sb::launch_heads_all<float>(p, T, vec, s) : sb::launch_heads_all<__nv_bfloat16>(p, T, vec, s);
}

extern "C" int sb_latent_place(const void* dq, const void* dkv, const void* q_norm, const void* kv_norm, const float* table,
                               const int* positions, const int* slots, void* q_out, void* cache, int T, int R1, int R2, int dims,
                               int interleaved, long dq_pitch, long dkv_pitch, float eps, int f32, cudaStream_t s) {
  if (T == 0) return 0;
  if (R1 <= 0 || R2 <= 0 || dims <= 0 || dims % 2) return (int)cudaErrorInvalidValue;
  const sb::LatentPlace a{dq, dkv, q_norm, kv_norm, table, positions, slots, q_out, cache, R1, R2, dims, interleaved, dq_pitch, dkv_pitch, eps};
  if (f32) return (int)sb::launch_pdl(sb::latent_place_kernel<float>, dim3(T), dim3(128), 0, s, a);
  return (int)sb::launch_pdl(sb::latent_place_kernel<__nv_bfloat16>, dim3(T), dim3(128), 0, s, a);
}

extern "C" int sb_latent_turn(const void* q, void* dst, const float* table, const int* positions, int T, int H, int D, int dims,
                              int interleaved, long q_pitch, long q_head, long dst_pitch, long dst_head, int f32, cudaStream_t s) {
  if (T == 0) return 0;
  if (H <= 0 || D < 0 || dims <= 0 || dims % 2) return (int)cudaErrorInvalidValue;
  const long pairs = static_cast<long>(T) * H * (dims / 2), want = (pairs + 255) / 256;
  const dim3 grid(static_cast<unsigned>(want < 148 * 16 ? want : 148 * 16));
  using bf16 = __nv_bfloat16;
  if (f32)
    return (int)sb::launch_pdl(sb::latent_turn_kernel<float>, grid, dim3(256), 0, s, (const float*)q, (float*)dst, table, positions, pairs, H,
                               D, dims, interleaved, q_pitch, q_head, dst_pitch, dst_head);
  return (int)sb::launch_pdl(sb::latent_turn_kernel<bf16>, grid, dim3(256), 0, s, (const bf16*)q, (bf16*)dst, table, positions, pairs, H, D,
                             dims, interleaved, q_pitch, q_head, dst_pitch, dst_head);
}

// Types: y_f32 / w_f32 (norm weights and h) = 1 for fp32, 0 for bf16; fp32 weights need fp32 y. H <= 8192. groups: parts of a row
// with an RMS norm of their own.
extern "C" int sb_stream_norm(const void* y, int y_f32, const int* ids, int y_rows, const int* dest, const float* wts, int k,
                              const void* shared, const float* gate, int gate_ld, const void* post_w, float* res, int init,
                              const void* pre_w, void* h, int w_f32, int T, int H, float eps, float w_off, int layer_norm,
                              const void* pair, const int* pair_ids, const int* prev, long mul_prev, long mul_cur, int pair_rows,
                              const float* plus, float h_scale, int groups, cudaStream_t s) {
  if (T == 0) return 0;
  if (groups < 1 || H % groups || (groups > 1 && layer_norm) || (pre_w != nullptr && h == nullptr)) return (int)cudaErrorInvalidValue;
  if (H <= 0 || H > sb::STREAM_MAX_H || (w_f32 && !y_f32) || (pair != nullptr && pair_rows <= 0)) return (int)cudaErrorInvalidValue;
  sb::StreamNorm a{y, ids, dest, wts, shared, gate, post_w, res, pre_w, h, k, y_rows, gate_ld, init, layer_norm, H, eps, w_off,
                   plus, h_scale, groups, pair, pair_ids, prev, mul_prev, mul_cur, pair_rows};
  bool vec = H % 8 == 0;
  for (const void* p : {y, pair, shared, post_w, static_cast<const void*>(plus), static_cast<const void*>(res), pre_w, static_cast<const void*>(h)})
    vec = vec && (reinterpret_cast<uintptr_t>(p) & 15) == 0;
  if (w_f32) return sb::launch_stream_norm<float, float>(a, T, vec, s);
  if (y_f32) return sb::launch_stream_norm<float, __nv_bfloat16>(a, T, vec, s);
  return sb::launch_stream_norm<__nv_bfloat16, __nv_bfloat16>(a, T, vec, s);
}

extern "C" int sb_glu(const void* in, const void* up, void* out, long rows, int F, long in_pitch, long out_pitch, int act, int f32,
                      cudaStream_t s) {
  if (rows == 0 || F == 0) return 0;
  if (act < 0 || act > 2) return (int)cudaErrorInvalidValue;
  const uintptr_t bits = reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(up) | reinterpret_cast<uintptr_t>(out);
  const bool vec = F % 8 == 0 && (bits & 15) == 0 && in_pitch % 8 == 0 && out_pitch % 8 == 0;
  const long n = rows * (vec ? F / 8 : F);
  const long want = (n + 255) / 256;
  const dim3 grid(static_cast<unsigned>(want < 148 * 16 ? want : 148 * 16)), block(256);
  using bf16 = __nv_bfloat16;
#define SB_GLU(T, V) \
  return (int)sb::launch_pdl(sb::glu_kernel<T, V>, grid, block, 0, s, (const T*)in, (const T*)up, (T*)out, rows, F, in_pitch, out_pitch, act)
  if (f32 && vec) SB_GLU(float, 8);
  if (f32) SB_GLU(float, 1);
  if (vec) SB_GLU(bf16, 8);
  SB_GLU(bf16, 1);
#undef SB_GLU
}

// in, out [T, F] (row pitches in_pitch, out_pitch); coef [4] fp32; sums [T, 3] or null, of rows of `all` units.
extern "C" int sb_poly_norm(const void* in, void* out, const float* coef, const float* sums, int T, int F, int all, long in_pitch,
                            long out_pitch, float eps, int f32, cudaStream_t s) {
  if (T == 0) return 0;
  if (F <= 0 || all < F) return (int)cudaErrorInvalidValue;
  const bool vec = F % 8 == 0 && ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(out)) & 15) == 0 && in_pitch % 8 == 0 && out_pitch % 8 == 0;
  using bf16 = __nv_bfloat16;
#define SB_POLY(T_, V) \
  return (int)sb::launch_pdl(sb::poly_norm_kernel<T_, V>, dim3(T), dim3(256), 0, s, (const T_*)in, (T_*)out, coef, sums, F, all, in_pitch, out_pitch, eps)
  if (f32 && vec) SB_POLY(float, 8);
  if (f32) SB_POLY(float, 1);
  if (vec) SB_POLY(bf16, 8);
  SB_POLY(bf16, 1);
#undef SB_POLY
}

// rows x n floats, rows `pitch` apart; rows <= 65535
extern "C" int sb_softcap(float* x, int rows, long n, long pitch, float cap, cudaStream_t s) {
  if (rows == 0 || n == 0) return 0;
  if (!(cap > 0.f) || rows > 65535) return (int)cudaErrorInvalidValue;
  const long want = (n + 1023) / 1024;
  return (int)sb::launch_pdl(sb::softcap_kernel, dim3(static_cast<unsigned>(want < 148 * 8 ? want : 148 * 8), rows), dim3(256), 0, s, x, n, pitch, cap);
}

// Row widths and pitches in bytes.
extern "C" int sb_kv_scatter(const void* k, const void* v, const int* slots, void* k_cache, void* v_cache, int T, int kb, int vb,
                             long k_pitch, long v_pitch, cudaStream_t s) {
  if (T == 0) return 0;
  const uintptr_t bits = reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(k_cache) |
                         reinterpret_cast<uintptr_t>(v_cache) | kb | vb | k_pitch | v_pitch;
  const char *kp = (const char*)k, *vp = (const char*)v;
  char *kc = (char*)k_cache, *vc = (char*)v_cache;
  if (bits % 16 == 0) return (int)sb::launch_pdl(sb::kv_scatter_kernel<uint4>, dim3(T), dim3(128), 0, s, kp, vp, slots, kc, vc, kb, vb, k_pitch, v_pitch);
  if (bits % 4 == 0) return (int)sb::launch_pdl(sb::kv_scatter_kernel<uint32_t>, dim3(T), dim3(128), 0, s, kp, vp, slots, kc, vc, kb, vb, k_pitch, v_pitch);
  if (bits % 2 == 0) return (int)sb::launch_pdl(sb::kv_scatter_kernel<uint16_t>, dim3(T), dim3(128), 0, s, kp, vp, slots, kc, vc, kb, vb, k_pitch, v_pitch);
  return (int)cudaErrorInvalidValue;
}
