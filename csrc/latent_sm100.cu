// Latent attention on the 5th-gen tensor cores (sm_100a): queries that have absorbed the key expansion, over the paged cache of
// latent vectors, and the per-head products around it.
//
// sb_latent_attn: one query token per CTA row, all heads share the cached vectors [c (R) | rotated key (W - R)]. Bound by
// streaming the cache once; a vector is key and value at the same time, so it is fetched once and used by both contractions:
//
//   TMA      64 tokens x W as 128-wide pairs of 64-wide chunks -> ring of pair buffers in smem (128B swizzle)
//   tcgen05  S^T[64 tok, HN] = C · Q^T      A = the tile (K-major), B = HN query heads
//   threads  one token per thread: its HN scores, tile max per head, exp, P^T -> smem (bf16)
//   tcgen05  O^T_b[128 dims, HN] = C_b^T · P^T   A = pair b of the tile read MN-major, one product per 128 value dims
//   threads  one output dim per thread and block: online-softmax merge in registers
//
// Warp 0 loads, warp 1 issues the products, warps 2-5 are the threads above. What has to be short is the chain from one
// tile's scores to the next one's, so scores, P^T and O^T have two buffers each: the scores of the next tile are formed under
// the softmax of this one (the ring holds at least two tiles), and a tile's O^T is merged after the next tile's P^T is out. The
// maximum is raised only when it has grown by 2^8, so most tiles rescale nothing. A pair that only holds key coordinates is
// released after the scores, value pairs with the products. The score
// product has 128 rows, of which the lower 64 are the tokens; the upper ones are whatever lies behind the chunk in shared
// memory and are never read.
// Grid = (rows, head groups, splits); with splits > 1 partial (o, m, l) go to a workspace and the combine kernel finishes.
//
// sb_head_gemm: C[:, h] = A[:, h] · B[h] (times sigmoid(gate)), every head one small product: 128 x 128 tiles (128 x 64 for few
// rows), 64-deep stages.
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

constexpr int LA_TILE = 64;
constexpr int LA_THREADS = 192;
constexpr int LA_CHUNK = LA_TILE * 128;  // bytes of 64 tokens x 64 elements
constexpr int LA_PAIR = 2 * LA_CHUNK;
constexpr int LA_MAX_RING = 13;
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
  constexpr int TMEM_COLS = 64 + 64 * NB <= 128 ? 128 : (64 + 64 * NB <= 256 ? 256 : 512);  // S @0, @32; O_b @64 + 32 b, + 32 NB
  extern __shared__ uint8_t smem_raw[];
  uint8_t* sR = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = sR + a.ring * LA_PAIR;
  uint8_t* sP = sQ + a.nchunk * (HN * 128);
  __shared__ uint64_t full[LA_MAX_RING], empty[LA_MAX_RING], s_full[2], p_full[2], o_full[2];
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_flag;
  __shared__ __align__(16) float red_m[2][HN][2];
  __shared__ float m_s[2][HN], red_l[4][HN];
  volatile int* cta_abort = &abort_flag;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x, h0 = blockIdx.y * HN, sp = blockIdx.z;
  if (threadIdx.x == 0) {
    for (int s = 0; s < a.ring; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(&s_full[b], 1);
      mbar_init(&p_full[b], 4);  // one arrival per softmax warp
      mbar_init(&o_full[b], 1);
    }
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
    // -------------------------------------------------------------- TMA producer (lane p: box p of the tile, a page or a part of one)
    const int rows = min(a.page_size, LA_TILE);  // of a box
    auto box_slot = [&](int i) {
      const int key = (tile0 + i) * LA_TILE + lane * rows;
      return i < n && lane * rows < LA_TILE && key < len ? bt[key >> a.page_shift] * a.page_size + (key & (a.page_size - 1)) : 0;
    };
    bool ok = true;
    int slot = box_slot(0);
    for (int i = 0, it = 0; i < n && ok; ++i) {
      const int next = box_slot(i + 1);
      const int boxes = (min(LA_TILE, len - (tile0 + i) * LA_TILE) + rows - 1) / rows;
      for (int p = 0; p < a.npair; ++p, ++it) {
        const int st = it % a.ring, chunks = min(2, a.nchunk - 2 * p);
        if (lane == 0) {
          ok = mbar_wait(&empty[st], (it / a.ring & 1) ^ 1, cta_abort, a.status, ERR_WAIT_EMPTY);
          if (ok) mbar_arrive_expect_tx(&full[st], boxes * rows * 128 * chunks);
        }
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (!ok) break;
        if (lane < boxes)
          for (int c = 0; c < chunks; ++c)
            tma_load_3d(sR + st * LA_PAIR + c * LA_CHUNK + lane * rows * 128, &tm, &full[st], (2 * p + c) * 64, 0, slot);
      }
      slot = next;
    }
  } else if (warp == 1) {
    // -------------------------------------------------------------- MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc(128, HN, 1, 1, 0, 0);
      constexpr uint32_t idesc_o = make_idesc(128, HN, 1, 1, 1, 0);  // A = the tile read MN-major
      const uint32_t r_addr = smem_u32(sR), q_addr = smem_u32(sQ), p_addr = smem_u32(sP);
      // Two sequences of work, whichever is ready first: pairs of the scores of tile ts (its buffer is free once the product of
      // tile ts - 2 has been issued), and the product of tile to. Waiting for one would hold up the other: copies for the scores
      // two tiles ahead only start when a product has released its pairs. One thread issues everything, so what it computes per
      // instruction counts: descriptors are sums (the address field is the lowest), ring positions are counters.
      const uint64_t ring_k = make_smem_desc(r_addr, 16, 1024, UMMA_SWIZZLE_128B), ring_v = make_smem_desc(r_addr, LA_CHUNK, 1024, UMMA_SWIZZLE_128B);
      const uint64_t desc_q = make_smem_desc(q_addr, 16, 1024, UMMA_SWIZZLE_128B), desc_p = make_smem_desc(p_addr, 16, 1024, UMMA_SWIZZLE_128B);
      int ts = 0, tp = 0, to = 0;
      int ss = 0, so = 0;  // ring positions of the next score pair and of the next product's first pair
      uint32_t full_par = 0;
      unsigned long long since = 0;
      for (uint32_t idle = 0; to < n;) {
        bool moved = false;
        if (to < ts && mbar_try_wait(&p_full[to & 1], to >> 1 & 1)) {
          tc_fence_after();
          const uint64_t dp = desc_p + (to & 1) * (HN * 128 / 16);
          const uint32_t d = tmem + 64 + (to & 1) * (32 * NB);
#pragma unroll
          for (int b = 0; b < NB; ++b) {
            const int st = so + b < a.ring ? so + b : so + b - a.ring;
            const uint64_t dv = ring_v + st * (LA_PAIR / 16);
#pragma unroll
            for (int k = 0; k < LA_TILE / 16; ++k) umma_f16(d + 32 * b, dv + k * (2048 / 16), dp + k * (32 / 16), idesc_o, k != 0 ? 1u : 0u);
            umma_commit(&empty[st]);
          }
          umma_commit(&o_full[to & 1]);
          so = so + a.npair < a.ring ? so + a.npair : so + a.npair - a.ring;
          ++to;
          moved = true;
        }
        if (ts < n && ts <= to + 1 && mbar_try_wait(&full[ss], full_par)) {
          tc_fence_after();
          const uint64_t dk = ring_k + ss * (LA_PAIR / 16), dq = desc_q + tp * (2 * HN * 128 / 16);
          const uint32_t d = tmem + 32 * (ts & 1);
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16(d, dk + k * (32 / 16), dq + k * (32 / 16), idesc_s, (tp | k) != 0 ? 1u : 0u);
          if (2 * tp + 1 < a.nchunk)
#pragma unroll
            for (int k = 0; k < 4; ++k) umma_f16(d, dk + (LA_CHUNK + k * 32) / 16, dq + (HN * 128 + k * 32) / 16, idesc_s, 1u);
          if (tp >= NB) umma_commit(&empty[ss]);
          if (++ss == a.ring) {
            ss = 0;
            full_par ^= 1;
          }
          if (++tp == a.npair) {
            umma_commit(&s_full[ts & 1]);
            tp = 0;
            ++ts;
          }
          moved = true;
        }
        if (moved) {
          idle = 0;
        } else if ((++idle & 0x3ff) == 0) {
          const unsigned long long now = globaltimer_ns();
          if (idle == 0x400) since = now;
          if (*cta_abort) break;
          if (now - since > WAIT_LIMIT_NS) {
            *cta_abort = 1;
            if (a.status) atomicCAS(a.status, 0, ERR_WAIT_FULL | (blockIdx.x << 8));
            break;
          }
        }
      }
    }
  } else {
    // -------------------------------------------------------------- softmax and merge
    const int quarter = warp & 3, tok = quarter * 32 + lane;  // TMEM lane = dim of a value block = token of the tile (if below 64)
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(quarter * 32) << 16);
    const float scale_log2 = a.rule.scale * 1.4426950408889634f;
    float acc[NB][HN], l_thr[HN];
#pragma unroll
    for (int g = 0; g < HN; ++g) {
      l_thr[g] = 0.f;
#pragma unroll
      for (int b = 0; b < NB; ++b) acc[b][g] = 0.f;
    }
    // acc <- acc + O^T of tile i: both in units of the maximum that tile i used
    auto merge = [&](int i, bool ok) {
      ok = ok && mbar_wait(&o_full[i & 1], i >> 1 & 1, cta_abort, a.status, ERR_WAIT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) return false;
      tc_fence_after();
#pragma unroll
      for (int b = 0; b < NB; ++b) {
        uint32_t r[32];
        tmem_ld_32x32(lane_addr + 64 + (i & 1) * (32 * NB) + 32 * b, r);
        tmem_ld_wait();
#pragma unroll
        for (int g = 0; g < HN; ++g) acc[b][g] += __uint_as_float(r[g]);
      }
      return true;
    };
    // maximum in use after a tile: raised only when it has grown a lot; the same in every thread
    auto raised = [&](int par, int g) {
      const float2 wm = *reinterpret_cast<const float2*>(red_m[par][g]);
      const float m_old = m_s[par][g], m_tile = fmaxf(wm.x, wm.y);
      return m_tile > m_old + 8.f ? m_tile : m_old;
    };
    bool ok = true;
    for (int i = 0; i < n; ++i) {  // every warp takes every turn: the barrier inside counts all of them, also after an expired wait
      const int par = i & 1, valid = min(LA_TILE, len - (tile0 + i) * LA_TILE);
      ok = ok && mbar_wait(&s_full[par], i >> 1 & 1, cta_abort, a.status, ERR_WAIT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      float sc[HN];
      if (quarter < 2) {  // these warps have the tokens
        uint32_t r[32];
        if (ok) {
          tc_fence_after();
          tmem_ld_32x32(lane_addr + 32 * par, r);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int g = 0; g < 32; ++g) r[g] = 0;
        }
#pragma unroll
        for (int g = 0; g < HN; ++g) {
          sc[g] = tok < valid ? __uint_as_float(r[g]) * scale_log2 : -INFINITY;
          const float wm = la_warp_max(sc[g]);
          if (lane == 0) red_m[par][g][quarter] = wm;
        }
      }
      softmax_warps_sync();
      if (quarter < 2) {
        uint8_t* p_col = sP + par * (HN * 128) + (tok & 7) * 2;
        const int piece = tok >> 3;
#pragma unroll
        for (int g = 0; g < HN; ++g) {
          const float m_old = m_s[par][g], m_use = raised(par, g);
          const float p = la_exp2(sc[g] - m_use);
          if (m_use != m_old) l_thr[g] *= la_exp2(m_old - m_use);
          l_thr[g] += p;
          *reinterpret_cast<__nv_bfloat16*>(p_col + g * 128 + ((piece ^ (g & 7)) << 4)) = __float2bfloat16(p);
        }
      }
      if (valid < LA_TILE && ok) {
        // Rows past the end hold whatever the page or an older tile left there: their p is 0, but 0 x NaN would poison O.
        // Every thread observes the copies' barriers before it overwrites a row.
#pragma unroll
        for (int b = 0; b < NB; ++b) {
          const int it = i * a.npair + b, st = it % a.ring;
          ok = ok && mbar_wait(&full[st], it / a.ring & 1, cta_abort, a.status, ERR_WAIT_FULL);
          if (ok && tok < LA_TILE && tok >= valid) {
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
      if (lane == 0 && ok) mbar_arrive(&p_full[par]);
      if (i > 0) ok = merge(i - 1, ok);
      bool any = false;
#pragma unroll
      for (int g = 0; g < HN; ++g) any |= raised(par, g) != m_s[par][g];
      if (any) {
#pragma unroll
        for (int g = 0; g < HN; ++g) {
          const float keep = la_exp2(m_s[par][g] - raised(par, g));
#pragma unroll
          for (int b = 0; b < NB; ++b) acc[b][g] *= keep;
        }
      }
      if (tok < HN) m_s[par ^ 1][tok] = raised(par, tok);
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
  // queries, P^T, alignment; the score product of the last chunk reads one chunk's bytes past the ring
  const int used = a.nchunk * HN * 128 + 2 * HN * 128, rest = (used > LA_CHUNK ? used : LA_CHUNK) + 1024;
  const int statics = 4 * 1024;  // barriers, maxima, sums
  a.ring = (LA_SMEM - statics - rest) / LA_PAIR;
  if (a.ring > LA_MAX_RING) a.ring = LA_MAX_RING;
  if (a.ring < 2 * a.npair) return -1;
  if (cudaError_t e = ensure_dynamic_smem(reinterpret_cast<const void*>(kern), LA_SMEM - statics); e != cudaSuccess) return (int)e;
  return (int)launch_pdl(kern, grid, dim3(LA_THREADS), a.ring * LA_PAIR + rest, s, tm, a);
}

// ------------------------------------------------------------------------------------------------- per-head products
constexpr int HG_BM = 128, HG_STAGES = 4;
template <int BN>
struct HgSmem {
  static constexpr int STAGE = (HG_BM + BN) * 128;  // 64 k of A and B
  static constexpr int TOTAL = HG_STAGES * STAGE + 1024;
};

struct HeadGemmArgs {
  __nv_bfloat16* c;
  const __nv_bfloat16* gate;
  int M, N, K;
  long c_row, c_head, gate_row, gate_head;
  int* status;
};

template <int BN, bool KN>  // KN: B stored [K, N]
__global__ void __launch_bounds__(192, 1)
head_gemm_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB, const __grid_constant__ HeadGemmArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  __shared__ uint64_t full[HG_STAGES], empty[HG_STAGES], done;
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_flag;
  volatile int* cta_abort = &abort_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = blockIdx.x * BN, m0 = blockIdx.y * HG_BM, h = blockIdx.z;
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
    tmem_alloc(&tmem_slot, BN);
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
      uint8_t* sA = smem + st * HgSmem<BN>::STAGE;
      uint8_t* sB = sA + HG_BM * 128;
      mbar_arrive_expect_tx(&full[st], HgSmem<BN>::STAGE);
      tma_load_3d(sA, &tmA, &full[st], k * 64, h, m0);
      if (KN) {  // chunks of 64 n, each 64 k rows
#pragma unroll
        for (int c = 0; c < BN / 64; ++c) tma_load_3d(sB + c * (64 * 128), &tmB, &full[st], n0 + c * 64, k * 64, h);
      } else {
        tma_load_3d(sB, &tmB, &full[st], k * 64, n0, h);
      }
    }
  } else if (warp == 1 && lane == 0) {
    constexpr uint32_t idesc = make_idesc(HG_BM, BN, 1, 1, 0, KN ? 1 : 0);
    bool ok = true;
    for (int k = 0; k < nk; ++k) {
      const int st = k % HG_STAGES;
      ok = mbar_wait(&full[st], k / HG_STAGES & 1, cta_abort, a.status, ERR_WAIT_FULL);
      if (!ok) break;
      tc_fence_after();
      const uint32_t sa = smem_u32(smem + st * HgSmem<BN>::STAGE), sb_ = sa + HG_BM * 128;
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
    const bool mine = m < a.M;
    constexpr int AHEAD = BN <= 64 ? BN / 8 : 1;  // few rows: the gate's values are fetched under the product
    uint4 gv[AHEAD];
    if (BN <= 64 && a.gate != nullptr && mine)
#pragma unroll
      for (int i = 0; i < AHEAD; ++i)
        if (n0 + i * 8 < a.N) gv[i] = *reinterpret_cast<const uint4*>(a.gate + m * a.gate_row + h * a.gate_head + n0 + i * 8);
    bool ok = mbar_wait(&done, 0, cta_abort, a.status, ERR_WAIT_TMEM_FULL);
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int c4 = 0; c4 < BN / 32; ++c4) {
        uint32_t r[32];
        tmem_ld_32x32(tmem + (static_cast<uint32_t>(quarter * 32) << 16) + c4 * 32, r);
        tmem_ld_wait();
        if (!mine) continue;
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
          const int n = n0 + c4 * 32 + i;
          if (n >= a.N) break;  // N is a multiple of 8
          float v[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) v[j] = __uint_as_float(r[i + j]);
          if (a.gate != nullptr) {
            const uint4 g = BN <= 64 ? gv[BN <= 64 ? c4 * 4 + i / 8 : 0] : *reinterpret_cast<const uint4*>(a.gate + m * a.gate_row + h * a.gate_head + n);
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
  if (warp == 1) tmem_dealloc(tmem, BN);
}

template <int BN, bool KN>
static int launch_head_gemm(int H, const CUtensorMap& ta, const CUtensorMap& tb, const HeadGemmArgs& a, cudaStream_t s) {
  auto kern = head_gemm_kernel<BN, KN>;
  if (cudaError_t e = ensure_dynamic_smem(reinterpret_cast<const void*>(kern), HgSmem<BN>::TOTAL); e != cudaSuccess) return (int)e;
  const dim3 grid((a.N + BN - 1) / BN, (a.M + HG_BM - 1) / HG_BM, H);
  return (int)launch_pdl(kern, grid, dim3(192), HgSmem<BN>::TOTAL, s, ta, tb, a);
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
  if (R > 512 || W > 640 || W % 8 || (heads != 16 && heads != 32) || splits > 32) return -1;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) & 15) return -1;
  try {
    const CUtensorMap tm = sb::make_tmap_3d(cache, W, 1, num_slots, W, W, 64, 1, page_size < sb::LA_TILE ? page_size : sb::LA_TILE);
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
  if ((M + sb::HG_BM - 1) / sb::HG_BM > 65535 || H > 65535) return -1;
  const bool few = M <= 256;  // then only narrow tiles occupy the machine
  const int bn = few ? 64 : 128;
  try {
    const CUtensorMap ta = sb::make_tmap_3d(A, K, H, M, a_head, a_row, 64, 1, sb::HG_BM);
    const CUtensorMap tb = b_kn ? sb::make_tmap_3d(B, N, K, H, b_ld, b_head, 64, 64, 1) : sb::make_tmap_3d(B, K, N, H, b_ld, b_head, 64, bn, 1);
    const sb::HeadGemmArgs a{(bf16*)C, (const bf16*)gate, M, N, K, c_row, c_head, gate_row, gate_head, status};
    if (few) return b_kn ? sb::launch_head_gemm<64, true>(H, ta, tb, a, s) : sb::launch_head_gemm<64, false>(H, ta, tb, a, s);
    return b_kn ? sb::launch_head_gemm<128, true>(H, ta, tb, a, s) : sb::launch_head_gemm<128, false>(H, ta, tb, a, s);
  } catch (const std::exception& e) {
    sb::set_last_error(e.what());
    return (int)cudaErrorInvalidValue;
  }
}
