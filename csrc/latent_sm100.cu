// Latent attention on the 5th-gen tensor cores (sm_100a): queries that have absorbed the key expansion, over the paged cache of
// latent vectors, and the per-head products around it.
//
// sb_latent_attn: one query token per CTA row, all heads share the cached vectors [c (R) | rotated key (W - R)]. Bound by
// streaming the cache once; a vector is key and value at the same time, so it is fetched once and used by both contractions:
//
//   TMA      128 tokens x W as 128-wide pairs of 64-wide chunks -> ring of pair buffers in smem (128B swizzle)
//   tcgen05  S^T[128 tok, HN] = C · Q^T     A = the tile (K-major), B = HN query heads
//   threads  one token per thread: its HN scores, tile max per head, exp, P^T -> smem (bf16)
//   tcgen05  O^T_b[128 dims, HN] = C_b^T · P^T   A = pair b of the tile read MN-major, one product per 128 value dims
//   threads  one output dim per thread and block: online-softmax merge in registers
//
// Warp 0 loads, warp 1 issues the products, warps 2-5 are the threads above. A pair that only holds key coordinates is
// released after the scores, value pairs one by one as their products finish, so the ring refills under the softmax.
// Grid = (rows, head groups, splits); with splits > 1 partial (o, m, l) go to a workspace and the combine kernel finishes.
//
// sb_head_gemm: C[:, h] = A[:, h] · B[h] (times sigmoid(gate)), every head one small product: 128 x 128 tiles, 64-deep stages.
//
// Every mbarrier wait is bounded: on expiry the CTA records a status word, skips its output, lets in-flight copies land, frees
// its TMEM and returns.
#include "attn_combine.cuh"

namespace sb {

__device__ __forceinline__ float la_exp2(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
__device__ __forceinline__ float la_warp_max(float v) {
  float r;
  asm volatile("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(r) : "f"(v));
  return r;
}
__device__ __forceinline__ void softmax_warps_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

constexpr int LA_TILE = 128;
constexpr int LA_THREADS = 192;
constexpr int LA_CHUNK = LA_TILE * 128;  // bytes of 128 tokens x 64 elements
constexpr int LA_PAIR = 2 * LA_CHUNK;
constexpr int LA_MAX_RING = 7;
constexpr int LA_SMEM = 227 * 1024;

struct LatentAttn {
  const __nv_bfloat16* q;  // [rows, H, W]
  const int *block_table, *row_req, *row_pos;
  __nv_bfloat16* out;  // [rows, H, R]
  float *part_o, *part_ml;
  int H, R, W, nchunk, npair, ring, page_size, page_shift, max_pages, splits;
  int* status;
  AttnRule rule;
};

// NB: 128-wide blocks of value dims; HN: query heads of a CTA
template <int NB, int HN>
__global__ void __launch_bounds__(LA_THREADS, 1)
latent_attn_kernel(const __grid_constant__ CUtensorMap tm, const __grid_constant__ LatentAttn a) {
  constexpr int TMEM_COLS = 32 + 32 * NB <= 128 ? 128 : 256;  // S @0, O_b @32 + 32 b
  extern __shared__ uint8_t smem_raw[];
  uint8_t* sR = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = sR + a.ring * LA_PAIR;
  uint8_t* sP = sQ + a.nchunk * (HN * 128);
  __shared__ uint64_t full[LA_MAX_RING], empty[LA_MAX_RING], s_full, p_full, o_full;
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_flag;
  __shared__ __align__(16) float red_m[2][HN][4];
  __shared__ float m_s[2][HN], red_l[4][HN];
  volatile int* cta_abort = &abort_flag;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x, h0 = blockIdx.y * HN, sp = blockIdx.z;
  if (threadIdx.x == 0) {
    for (int s = 0; s < a.ring; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(&s_full, 1);
    mbar_init(&p_full, 4);  // one arrival per softmax warp
    mbar_init(&o_full, 1);
    abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tm);
  }
  if (threadIdx.x < HN) m_s[0][threadIdx.x] = -INFINITY;
  if (warp == 1) {
    tmem_alloc(&tmem_slot, TMEM_COLS);
    tmem_relinquish();
  }
  pdl_wait();
  pdl_launch_dependents();
  const int len = a.row_pos[t] + 1;
  const int* bt = a.block_table + static_cast<size_t>(a.row_req != nullptr ? a.row_req[t] : t) * a.max_pages;
  const int total = (len + LA_TILE - 1) / LA_TILE, per = (total + a.splits - 1) / a.splits;
  const int tile0 = min(sp * per, total), n = min(total, tile0 + per) - tile0;
  // query heads, K-major 128B swizzle: 16-byte piece j of row r sits at j ^ (r % 8); surplus rows and columns are zero
  for (int i = threadIdx.x; i < HN * a.nchunk * 8; i += LA_THREADS) {
    const int j = i % 8, c = (i / 8) % a.nchunk, r = i / (8 * a.nchunk);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (h0 + r < a.H && c * 64 + j * 8 < a.W)
      v = *reinterpret_cast<const uint4*>(a.q + (static_cast<size_t>(t) * a.H + h0 + r) * a.W + c * 64 + j * 8);
    *reinterpret_cast<uint4*>(sQ + c * (HN * 128) + r * 128 + ((j ^ (r & 7)) << 4)) = v;
  }
  fence_proxy_async();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;

  if (warp == 0) {
    // -------------------------------------------------------------- TMA producer (lane p: page p of the tile)
    auto page_slot = [&](int i) {
      const int page = ((tile0 + i) * LA_TILE >> a.page_shift) + lane;
      return i < n && lane < (LA_TILE >> a.page_shift) && page << a.page_shift < len ? bt[page] * a.page_size : 0;
    };
    bool ok = true;
    int slot = page_slot(0);
    for (int i = 0, it = 0; i < n && ok; ++i) {
      const int next = page_slot(i + 1);
      const int npages = (min(LA_TILE, len - (tile0 + i) * LA_TILE) + a.page_size - 1) >> a.page_shift;
      for (int p = 0; p < a.npair; ++p, ++it) {
        const int st = it % a.ring, chunks = min(2, a.nchunk - 2 * p);
        if (lane == 0) {
          ok = mbar_wait(&empty[st], (it / a.ring & 1) ^ 1, cta_abort, a.status, ERR_WAIT_EMPTY);
          if (ok) mbar_arrive_expect_tx(&full[st], npages * a.page_size * 128 * chunks);
        }
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (!ok) break;
        if (lane < npages)
          for (int c = 0; c < chunks; ++c)
            tma_load_3d(sR + st * LA_PAIR + c * LA_CHUNK + lane * a.page_size * 128, &tm, &full[st], (2 * p + c) * 64, 0, slot);
      }
      slot = next;
    }
  } else if (warp == 1) {
    // -------------------------------------------------------------- MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc(LA_TILE, HN, 1, 1, 0, 0);
      constexpr uint32_t idesc_o = make_idesc(128, HN, 1, 1, 1, 0);  // A = the tile read MN-major
      const uint32_t r_addr = smem_u32(sR), q_addr = smem_u32(sQ), p_addr = smem_u32(sP);
      bool ok = true;
      for (int i = 0; i < n && ok; ++i) {
        const int it0 = i * a.npair;
        for (int p = 0; p < a.npair && ok; ++p) {
          const int st = (it0 + p) % a.ring, chunks = min(2, a.nchunk - 2 * p);
          ok = mbar_wait(&full[st], (it0 + p) / a.ring & 1, cta_abort, a.status, ERR_WAIT_FULL);
          if (!ok) break;
          tc_fence_after();
          for (int c = 0; c < chunks; ++c)
#pragma unroll
            for (int k = 0; k < 4; ++k)
              umma_f16(tmem, make_smem_desc(r_addr + st * LA_PAIR + c * LA_CHUNK + k * 32, 16, 1024, UMMA_SWIZZLE_128B),
                       make_smem_desc(q_addr + (2 * p + c) * (HN * 128) + k * 32, 16, 1024, UMMA_SWIZZLE_128B), idesc_s, (p | c | k) != 0 ? 1u : 0u);
          if (p >= NB) umma_commit(&empty[st]);
        }
        if (!ok) break;
        umma_commit(&s_full);
        ok = mbar_wait(&p_full, i & 1, cta_abort, a.status, ERR_WAIT_TMEM_EMPTY);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int b = 0; b < NB; ++b) {
          const int st = (it0 + b) % a.ring;
#pragma unroll
          for (int k = 0; k < LA_TILE / 16; ++k)
            umma_f16(tmem + 32 + 32 * b, make_smem_desc(r_addr + st * LA_PAIR + k * 2048, LA_CHUNK, 1024, UMMA_SWIZZLE_128B),
                     make_smem_desc(p_addr + (k >> 2) * (HN * 128) + (k & 3) * 32, 16, 1024, UMMA_SWIZZLE_128B), idesc_o, k != 0 ? 1u : 0u);
          umma_commit(&empty[st]);
        }
        umma_commit(&o_full);
      }
    }
  } else {
    // -------------------------------------------------------------- softmax and merge
    const int quarter = warp & 3, tok = quarter * 32 + lane;  // token of the tile = dim of a value block = TMEM lane
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(quarter * 32) << 16);
    const float scale_log2 = a.rule.scale * 1.4426950408889634f;
    float acc[NB][HN], l_thr[HN];
#pragma unroll
    for (int g = 0; g < HN; ++g) {
      l_thr[g] = 0.f;
#pragma unroll
      for (int b = 0; b < NB; ++b) acc[b][g] = 0.f;
    }
    // acc <- (acc + O^T of tile i): both in units of the maximum that tile i used
    auto merge = [&](int i, bool ok) {
      ok = ok && mbar_wait(&o_full, i & 1, cta_abort, a.status, ERR_WAIT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) return false;
      tc_fence_after();
#pragma unroll
      for (int b = 0; b < NB; ++b) {
        uint32_t r[32];
        tmem_ld_32x32(lane_addr + 32 + 32 * b, r);
        tmem_ld_wait();
#pragma unroll
        for (int g = 0; g < HN; ++g) acc[b][g] += __uint_as_float(r[g]);
      }
      return true;
    };
    bool ok = true;
    for (int i = 0; i < n; ++i) {  // every warp takes every turn: the barrier inside counts all of them, also after an expired wait
      const int par = i & 1, valid = min(LA_TILE, len - (tile0 + i) * LA_TILE);
      ok = ok && mbar_wait(&s_full, par, cta_abort, a.status, ERR_WAIT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      float sc[HN];
      {
        uint32_t r[32];
        if (ok) {
          tc_fence_after();
          tmem_ld_32x32(lane_addr, r);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int g = 0; g < 32; ++g) r[g] = 0;
        }
#pragma unroll
        for (int g = 0; g < HN; ++g) sc[g] = tok < valid ? __uint_as_float(r[g]) * scale_log2 : -INFINITY;
      }
#pragma unroll
      for (int g = 0; g < HN; ++g) {
        const float wm = la_warp_max(sc[g]);
        if (lane == 0) red_m[par][g][quarter] = wm;
      }
      softmax_warps_sync();
      if (i > 0) ok = merge(i - 1, ok);  // also frees P^T
      uint8_t* p_col = sP + (tok >> 6) * (HN * 128) + (tok & 7) * 2;
      const int piece = (tok & 63) >> 3;
#pragma unroll
      for (int g = 0; g < HN; ++g) {
        const float4 wm = *reinterpret_cast<const float4*>(red_m[par][g]);
        const float m_old = m_s[par][g];
        const float m_new = fmaxf(m_old, fmaxf(fmaxf(wm.x, wm.y), fmaxf(wm.z, wm.w)));  // the same in every thread
        const float keep = la_exp2(m_old - m_new);
        const float p = la_exp2(sc[g] - m_new);
        l_thr[g] = l_thr[g] * keep + p;
#pragma unroll
        for (int b = 0; b < NB; ++b) acc[b][g] *= keep;
        if (tok == g) m_s[par ^ 1][g] = m_new;
        *reinterpret_cast<__nv_bfloat16*>(p_col + g * 128 + ((piece ^ (g & 7)) << 4)) = __float2bfloat16(p);
      }
      if (valid < LA_TILE && ok) {
        // Rows past the end hold whatever the page or an older tile left there: their p is 0, but 0 x NaN would poison O.
        // Every thread observes the copies' barriers before it overwrites a row.
#pragma unroll
        for (int b = 0; b < NB; ++b) {
          const int it = i * a.npair + b, st = it % a.ring;
          ok = ok && mbar_wait(&full[st], it / a.ring & 1, cta_abort, a.status, ERR_WAIT_FULL);
          if (ok && tok >= valid) {
            uint4* row = reinterpret_cast<uint4*>(sR + st * LA_PAIR + tok * 128);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
              row[j] = make_uint4(0, 0, 0, 0);
              row[LA_CHUNK / 16 + j] = make_uint4(0, 0, 0, 0);
            }
          }
        }
      }
      fence_proxy_async();
      tc_fence_before();
      ok = __all_sync(0xffffffffu, ok);
      if (lane == 0 && ok) mbar_arrive(&p_full);
    }
    if (n > 0) ok = merge(n - 1, ok);
#pragma unroll
    for (int g = 0; g < HN; ++g) {
      const float ws = warp_sum(l_thr[g]);
      if (lane == 0) red_l[quarter][g] = ws;
    }
    softmax_warps_sync();
    if (ok && *cta_abort == 0) {
#pragma unroll
      for (int g = 0; g < HN; ++g) {
        if (h0 + g >= a.H) break;
        const float l = red_l[0][g] + red_l[1][g] + red_l[2][g] + red_l[3][g];
        const size_t row = static_cast<size_t>(t) * a.H + h0 + g;
        const float inv = a.splits > 1 ? 1.f : (l > 0.f ? a.rule.out_scale / l : 0.f);
#pragma unroll
        for (int b = 0; b < NB; ++b) {
          const int d = b * 128 + tok;
          if (d >= a.R) continue;
          if (a.splits > 1) a.part_o[(row * a.splits + sp) * a.R + d] = acc[b][g];
          else a.out[row * a.R + d] = __float2bfloat16(acc[b][g] * inv);
        }
        if (a.splits > 1 && tok == 0) {
          a.part_ml[(row * a.splits + sp) * 2] = m_s[n & 1][g] * 0.6931471805599453f;  // natural logarithms from here on
          a.part_ml[(row * a.splits + sp) * 2 + 1] = l;
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (*cta_abort) {
    const unsigned long long t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);  // let copies in flight land
    __syncthreads();
  }
  if (warp == 1) tmem_dealloc(tmem, TMEM_COLS);
}

template <int NB, int HN>
static int launch_latent_attn(dim3 grid, const CUtensorMap& tm, LatentAttn a, cudaStream_t s) {
  auto kern = latent_attn_kernel<NB, HN>;
  const int rest = a.nchunk * HN * 128 + 2 * HN * 128 + 1024;  // queries, P^T, alignment
  const int statics = 4 * 1024;  // barriers, maxima, sums
  a.ring = (LA_SMEM - statics - rest) / LA_PAIR;
  if (a.ring > LA_MAX_RING) a.ring = LA_MAX_RING;
  if (a.ring < a.npair) return -1;
  if (cudaError_t e = ensure_dynamic_smem(reinterpret_cast<const void*>(kern), LA_SMEM - statics); e != cudaSuccess) return (int)e;
  return (int)launch_pdl(kern, grid, dim3(LA_THREADS), a.ring * LA_PAIR + rest, s, tm, a);
}

// ------------------------------------------------------------------------------------------------- per-head products
constexpr int HG_BM = 128, HG_BN = 128, HG_STAGES = 4;
constexpr int HG_STAGE = (HG_BM + HG_BN) * 128;  // 64 k of A and B
constexpr int HG_SMEM = HG_STAGES * HG_STAGE + 1024;

struct HeadGemmArgs {
  __nv_bfloat16* c;
  const __nv_bfloat16* gate;
  int M, N, K;
  long c_row, c_head, gate_row, gate_head;
  int* status;
};

template <bool KN>  // B stored [K, N]
__global__ void __launch_bounds__(192, 1)
head_gemm_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB, const __grid_constant__ HeadGemmArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  __shared__ uint64_t full[HG_STAGES], empty[HG_STAGES], done;
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_flag;
  volatile int* cta_abort = &abort_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = blockIdx.x * HG_BN, m0 = blockIdx.y * HG_BM, h = blockIdx.z;
  const int nk = (a.K + 63) / 64;
  if (threadIdx.x == 0) {
    for (int s = 0; s < HG_STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(&done, 1);
    abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tmA);
    tma_prefetch_desc(&tmB);
  }
  if (warp == 1) {
    tmem_alloc(&tmem_slot, HG_BN);
    tmem_relinquish();
  }
  pdl_wait();
  pdl_launch_dependents();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  if (warp == 0 && lane == 0) {
    for (int k = 0; k < nk; ++k) {
      const int st = k % HG_STAGES;
      if (!mbar_wait(&empty[st], (k / HG_STAGES & 1) ^ 1, cta_abort, a.status, ERR_WAIT_EMPTY)) break;
      uint8_t* sA = smem + st * HG_STAGE;
      uint8_t* sB = sA + HG_BM * 128;
      mbar_arrive_expect_tx(&full[st], HG_STAGE);
      tma_load_3d(sA, &tmA, &full[st], k * 64, h, m0);
      if (KN) {  // two chunks of 64 n, each 64 k rows
        tma_load_3d(sB, &tmB, &full[st], n0, k * 64, h);
        tma_load_3d(sB + 64 * 128, &tmB, &full[st], n0 + 64, k * 64, h);
      } else {
        tma_load_3d(sB, &tmB, &full[st], k * 64, n0, h);
      }
    }
  } else if (warp == 1 && lane == 0) {
    constexpr uint32_t idesc = make_idesc(HG_BM, HG_BN, 1, 1, 0, KN ? 1 : 0);
    bool ok = true;
    for (int k = 0; k < nk; ++k) {
      const int st = k % HG_STAGES;
      ok = mbar_wait(&full[st], k / HG_STAGES & 1, cta_abort, a.status, ERR_WAIT_FULL);
      if (!ok) break;
      tc_fence_after();
      const uint32_t sa = smem_u32(smem + st * HG_STAGE), sb_ = sa + HG_BM * 128;
#pragma unroll
      for (int j = 0; j < 4; ++j)
        umma_f16(tmem, make_smem_desc(sa + j * 32, 16, 1024, UMMA_SWIZZLE_128B),
                 KN ? make_smem_desc(sb_ + j * 2048, 64 * 128, 1024, UMMA_SWIZZLE_128B) : make_smem_desc(sb_ + j * 32, 16, 1024, UMMA_SWIZZLE_128B),
                 idesc, (k | j) != 0 ? 1u : 0u);
      umma_commit(&empty[st]);
    }
    if (ok) umma_commit(&done);
  } else if (warp >= 2) {
    const int quarter = warp & 3, m = m0 + quarter * 32 + lane;
    bool ok = mbar_wait(&done, 0, cta_abort, a.status, ERR_WAIT_TMEM_FULL);
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int c4 = 0; c4 < HG_BN / 32; ++c4) {
        uint32_t r[32];
        tmem_ld_32x32(tmem + (static_cast<uint32_t>(quarter * 32) << 16) + c4 * 32, r);
        tmem_ld_wait();
        if (m >= a.M) continue;
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
          const int n = n0 + c4 * 32 + i;
          if (n >= a.N) break;  // N is a multiple of 8
          float v[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) v[j] = __uint_as_float(r[i + j]);
          if (a.gate != nullptr) {
            const uint4 g = *reinterpret_cast<const uint4*>(a.gate + m * a.gate_row + h * a.gate_head + n);
            const uint32_t gs[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              const float2 z = unpack_bf16x2(gs[j]);
              v[2 * j] *= sigmoid_f(z.x);
              v[2 * j + 1] *= sigmoid_f(z.y);
            }
          }
          *reinterpret_cast<uint4*>(a.c + m * a.c_row + h * a.c_head + n) =
              make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (*cta_abort) {
    const unsigned long long t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);  // let copies in flight land
    __syncthreads();
  }
  if (warp == 1) tmem_dealloc(tmem, HG_BN);
}

}  // namespace sb

// q [T, H, W] bf16 contiguous; cache [num_slots, W] bf16, of which the first R elements are the value; row t sees positions
// 0 .. row_pos[t] of request row_req[t] (null: request t); out [T, H, R] contiguous; part_o [T, H, splits, R] and part_ml
// [T, H, splits, 2] fp32 workspaces, used when splits > 1. heads: query heads of a CTA, 16 or 32.
// Returns 0, a cudaError_t value, or -1 for what the kernel does not take (R above 512, W above 640, widths no multiple of 8).
extern "C" int sb_latent_attn(const void* q, const void* cache, const int* block_table, const int* row_req, const int* row_pos, void* out,
                              float* part_o, float* part_ml, int T, int H, int R, int W, int page_size, int max_pages, int num_slots,
                              int heads, int splits, const void* attn_rule, int* status, cudaStream_t s) {
  using bf16 = __nv_bfloat16;
  const sb::AttnRule* rule = (const sb::AttnRule*)attn_rule;
  if (T == 0) return 0;
  if (H <= 0 || R <= 0 || W < R || splits < 1 || !rule_ok(rule)) return (int)cudaErrorInvalidValue;
  int shift = 0;
  while ((1 << shift) < page_size) ++shift;
  if ((1 << shift) != page_size || page_size < 16 || page_size > 128) return -1;
  if (R > 512 || W > 640 || W % 8 || (heads != 16 && heads != 32)) return -1;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) & 15) return -1;
  try {
    const CUtensorMap tm = sb::make_tmap_3d(cache, W, 1, num_slots, W, W, 64, 1, page_size);
    const int nchunk = (W + 63) / 64;
    const sb::LatentAttn a{(const bf16*)q, block_table, row_req, row_pos, (bf16*)out, part_o, part_ml, H, R, W, nchunk, (nchunk + 1) / 2, 0,
                           page_size, shift, max_pages, splits, status, *rule};
    const dim3 grid(T, (H + heads - 1) / heads, splits);
    const int nb = (R + 127) / 128;
    int rc = -1;
#define SB_LA(NB)                                                                                               \
  if (nb == NB) rc = heads == 16 ? sb::launch_latent_attn<NB, 16>(grid, tm, a, s) : sb::launch_latent_attn<NB, 32>(grid, tm, a, s);
    SB_LA(1) SB_LA(2) SB_LA(3) SB_LA(4)
#undef SB_LA
    if (rc != 0) return rc;
    if (splits > 1)
      return (int)sb::launch_pdl(sb::attn_combine_kernel, dim3(T * H), dim3(R <= 128 ? 64 : 128), 0, s, part_o, part_ml, (bf16*)out, R, R,
                                 splits, H * R, H, *rule);
    return (int)cudaGetLastError();
  } catch (const std::exception& e) {
    sb::set_last_error(e.what());
    return (int)cudaErrorInvalidValue;
  }
}

// C[m, h, n] = sigmoid(gate[m, h, n]) * sum_k A[m, h, k] B[h][n, k] (B stored [N, K], or [K, N] with b_kn), bf16, pitches in elements.
// Returns -1 for widths that are no multiple of 8 or misaligned operands.
extern "C" int sb_head_gemm(const void* A, const void* B, void* C, const void* gate, int H, int M, int N, int K, int b_kn, long a_row,
                            long a_head, long b_head, long b_ld, long c_row, long c_head, long gate_row, long gate_head, int* status,
                            cudaStream_t s) {
  using bf16 = __nv_bfloat16;
  if (H <= 0 || M <= 0 || N <= 0) return 0;
  if (K <= 0) return (int)cudaErrorInvalidValue;
  if (N % 8 || K % 8 || a_row % 8 || a_head % 8 || b_head % 8 || b_ld % 8 || c_row % 8 || c_head % 8 || gate_row % 8 || gate_head % 8) return -1;
  if ((reinterpret_cast<uintptr_t>(A) | reinterpret_cast<uintptr_t>(B) | reinterpret_cast<uintptr_t>(C) | reinterpret_cast<uintptr_t>(gate)) & 15)
    return -1;
  const dim3 grid((N + sb::HG_BN - 1) / sb::HG_BN, (M + sb::HG_BM - 1) / sb::HG_BM, H);
  if (grid.y > 65535 || grid.z > 65535) return -1;
  try {
    const CUtensorMap ta = sb::make_tmap_3d(A, K, H, M, a_head, a_row, 64, 1, sb::HG_BM);
    const CUtensorMap tb = b_kn ? sb::make_tmap_3d(B, N, K, H, b_ld, b_head, 64, 64, 1) : sb::make_tmap_3d(B, K, N, H, b_ld, b_head, 64, sb::HG_BN, 1);
    const sb::HeadGemmArgs a{(bf16*)C, (const bf16*)gate, M, N, K, c_row, c_head, gate_row, gate_head, status};
    auto kern = b_kn ? sb::head_gemm_kernel<true> : sb::head_gemm_kernel<false>;
    if (cudaError_t e = sb::ensure_dynamic_smem(reinterpret_cast<const void*>(kern), sb::HG_SMEM); e != cudaSuccess) return (int)e;
    return (int)sb::launch_pdl(kern, grid, dim3(192), sb::HG_SMEM, s, ta, tb, a);
  } catch (const std::exception& e) {
    sb::set_last_error(e.what());
    return (int)cudaErrorInvalidValue;
  }
}
