// Attention of prompt rows over the paged KV cache, on the 5th-gen tensor cores (sm_100a). Sister of
// flash_fwd_sm100.cu (same warp roles, same softmax scheme) for layers whose queries see a sliding window plus the first
// tokens of the sequence, or the keys of their own chunk, and whose scores are capped or depend on the distance:
// attn_rule.cuh has the equations.
//
// Eight softmax warps work on a tile, two on every scheduler: one group of four has the first 64 keys of every tile, the other
// the last 64. The groups share nothing but the score tile: each has its own running maximum, sum and output accumulator, as
// if the keys were split between two launches, and the epilogue joins the two.
//
// Two more things differ in structure. Keys and values come straight from the cache pages (one TMA box per page and 64-wide
// chunk), so a later portion of a prompt, portions of several requests and single tokens beside them are one launch without
// a gather. And the G = Hq / Hkv query heads of a kv head are stacked into the rows of one tile (row = token * G + head), so
// every key tile is loaded once for all of them and a single token still fills G rows.
//
// Work comes from a table built on the host: tile t = (first row of q, tokens, position of the first token, request). A CTA
// visits only key tiles that some row of its tile can see: the tiles that hold the kept first tokens, then 128-key tiles
// from the page that holds the first key of the window up to the last token. Rows with nothing visible yet keep a running
// maximum of -inf; the first tile that shows them a key corrects it like any later rise.
//
// The distance penalty costs the softmax nothing per element. Inside a key tile it is slope * (key0 - i) + slope * c for
// column c: the first term is one number per row and tile, the second is one more k-step of the score product, with
// (hi, mid, lo) of slope / scale in the row's three extra query columns and (c, c, c) in the extra key columns. The three
// bf16 parts carry all 24 bits of the factor, c <= 127 is exact, and the extra key columns are the same for every tile.
//
// Capped scores and learned distance biases (RULED) need every score before its maximum, so a row's 128 scores stay in
// registers. tanh costs an exponential and half a reciprocal (two scores share one). The bias of a tile whose keys are all
// far is one number per row; elsewhere it comes from a table by distance in shared memory, [distance][head of the group]:
// row r = token * G + head reads entry (distance of column 0) * G + r - c * G, so a warp's reads are adjacent.
//
// Keys may come in two parts (latent attention): the first `kchunks` 64-wide chunks from one tensor per head, the others from
// a second one that all heads share, and queries likewise. Keys wider than 128 leave room for one value stage only.
// Pairs of heads (FORM 2): the two attentions of an output head are adjacent rows of the tile, so adjacent lanes exchange their columns
// in the epilogue; the two groups of warps, which have half of the columns each, exchange the sum of squares.
#include "attn_rule.cuh"

namespace sb {

enum : int { FW_PLAIN = 0, FW_RULED = 1, FW_PAIR = 2 };
constexpr int FW_BM = 128, FW_BN = 128;
constexpr int FW_HALF = FW_BN / 2;  // keys of a tile per softmax group
constexpr int FW_THREADS = 320;     // TMA warp, MMA warp, 2 groups of 4 softmax warps
constexpr int FW_STAGES = 2;

template <int DK, int DV>
struct FwSmem {
  static constexpr int VSTAGES = DK > 128 ? 1 : 2;
  static constexpr int KCH = DK / 64, VCH = DV / 64;
  static constexpr int Q_BYTES = FW_BM * 128 * KCH;
  static constexpr int K_BYTES = FW_BN * 128 * KCH;
  static constexpr int V_BYTES = FW_BN * 128 * VCH;
  static constexpr int P_BYTES = FW_BM * FW_BN * 2;
  // extra columns of the distance penalty (k-step 0 of row r = query row r's, k-step 1 = key column r's), or bias by distance
  static constexpr int X_BYTES = DK > 128 ? 0 : FW_BM * 128;
  static constexpr int TOTAL = Q_BYTES + FW_STAGES * K_BYTES + VSTAGES * V_BYTES + P_BYTES + X_BYTES + 256 + 1024;  // + barriers, alignment
  static constexpr int TMEM_COLS = 512;  // S0 @0, S1 @128, O of the first group @256, of the second @256 + DV
};

__device__ __forceinline__ float fw_exp2(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

// The n lowest bits (n <= 0: none, n >= 32: all).
__device__ __forceinline__ uint32_t fw_below(int n) {
  return n <= 0 ? 0u : (n >= 32 ? 0xffffffffu : (1u << n) - 1);
}

struct FwArgs {
  const int* block_table;
  const int4* tiles;
  __nv_bfloat16* out;
  int Hq, Hkv, G, dv, page_size, page_shift, max_pages;
  int kchunks;  // chunks of a key (and query) that come from the first tensor of each pair
  long out_stride;
  int* status;
  AttnRule rule;
};

template <int DK, int DV, int FORM>
__global__ void __launch_bounds__(FW_THREADS, 1)
flash_window_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                    const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmQ2,
                    const __grid_constant__ CUtensorMap tmK2, const __grid_constant__ FwArgs a) {
  using S = FwSmem<DK, DV>;
  constexpr bool RULED = FORM == FW_RULED, PAIR = FORM == FW_PAIR;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + S::Q_BYTES;
  uint8_t* sV = sK + FW_STAGES * S::K_BYTES;
  uint8_t* sP = sV + S::VSTAGES * S::V_BYTES;
  uint8_t* sX = sP + S::P_BYTES;
  uint64_t* q_full = reinterpret_cast<uint64_t*>(sX + S::X_BYTES);
  uint64_t* k_full = q_full + 1;
  uint64_t* k_empty = k_full + FW_STAGES;
  uint64_t* v_full = k_empty + FW_STAGES;
  uint64_t* v_empty = v_full + FW_STAGES;
  uint64_t* s_full = v_empty + FW_STAGES;  // [2]
  uint64_t* p_full = s_full + 2;  // [2]
  uint64_t* o_done = p_full + 2;  // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 2);
  volatile int* cta_abort = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* status = a.status;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kvh = blockIdx.y;
  const int G = a.G, bq = FW_BM / G;  // heads and tokens of a tile

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < FW_STAGES; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1);
      mbar_init(&v_empty[s], 1);
    }
    mbar_init(&s_full[0], 1);
    mbar_init(&s_full[1], 1);
    for (int g = 0; g < 2; ++g) {
      mbar_init(&p_full[g], 4);  // one arrival per softmax warp
      mbar_init(&o_done[g], 1);
    }
    *cta_abort = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
    if (a.kchunks < S::KCH) {
      tma_prefetch_desc(&tmQ2);
      tma_prefetch_desc(&tmK2);
    }
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, S::TMEM_COLS);
    tmem_relinquish();
  }
  pdl_wait();
  pdl_launch_dependents();
  // RULED: bias by distance times log2 e, in shared memory when it fits
  const int far = a.rule.bias_rows - 1;
  const bool near_table = RULED && a.rule.bias != nullptr && a.rule.bias_rows * G * 4 <= S::X_BYTES;
  if (near_table && warp >= 2) {
    float* tab = reinterpret_cast<float*>(sX);
    for (int i = threadIdx.x - 64; i < a.rule.bias_rows * G; i += 256)
      tab[i] = a.rule.bias[static_cast<size_t>(i / G) * a.Hq + kvh * G + i % G] * 1.4426950408889634f;
  }
  if (!RULED && S::X_BYTES > 0 && a.rule.slopes != nullptr && warp >= 2 && warp < 6) {
    const int r = threadIdx.x - 64;
    const float f = r < bq * G ? a.rule.slopes[kvh * G + r % G] / a.rule.scale : 0.f;
    const __nv_bfloat16 hi = __float2bfloat16(f);
    const float f1 = f - __bfloat162float(hi);
    const __nv_bfloat16 mid = __float2bfloat16(f1);
    const float f2 = f1 - __bfloat162float(mid);
    const float c = static_cast<float>(r);
    uint8_t* x = sX + r * 128;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    *reinterpret_cast<uint4*>(x + ((0 ^ (r & 7)) << 4)) =
        make_uint4(pack_bf16x2(__bfloat162float(hi), __bfloat162float(mid)), pack_bf16x2(f2, 0.f), 0, 0);
    *reinterpret_cast<uint4*>(x + ((1 ^ (r & 7)) << 4)) = zero;
    *reinterpret_cast<uint4*>(x + ((2 ^ (r & 7)) << 4)) = make_uint4(pack_bf16x2(c, c), pack_bf16x2(c, 0.f), 0, 0);
    *reinterpret_cast<uint4*>(x + ((3 ^ (r & 7)) << 4)) = zero;
    fence_proxy_async();  // plain stores -> visible to the tensor core
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  const int4 work = a.tiles[blockIdx.x];
  const int row0 = work.x, ntok = work.y, p0 = work.z;
  const int* bt = a.block_table + static_cast<size_t>(work.w) * a.max_pages;
  const int hi = p0 + ntok;                                         // keys [0, hi) exist
  const int lo = rule_first_key(a.rule, p0);                        // first key of the first row's window or chunk
  int base = (lo >> a.page_shift) << a.page_shift;                  // windowed tiles start at a page
  const int n_keep = min((min(a.rule.keep_first, hi) + FW_BN - 1) / FW_BN, (base + FW_BN - 1) / FW_BN);
  base = max(base, n_keep * FW_BN);
  const int n_kv = n_keep + (hi > base ? (hi - base + FW_BN - 1) / FW_BN : 0);
  auto key0_of = [&](int j) { return j < n_keep ? j * FW_BN : base + (j - n_keep) * FW_BN; };

  if (warp == 0) {
    // -------------------------------------------------------------------- TMA producer (lane p: page p of the tile)
    if (lane == 0) {
      mbar_arrive_expect_tx(q_full, bq * G * 128 * S::KCH);
#pragma unroll
      for (int c = 0; c < S::KCH; ++c) {
        if (c < a.kchunks) tma_load_3d(sQ + c * (FW_BM * 128), &tmQ, q_full, c * 64, kvh * G, row0);
        else tma_load_3d(sQ + c * (FW_BM * 128), &tmQ2, q_full, (c - a.kchunks) * 64, kvh * G, row0);
      }
    }
    // keys run one tile ahead of the values, whose buffer is free only once the product of an earlier tile is done
    bool ok = true;
    int slot_k = 0;
    for (int j = 0; j <= n_kv && ok; ++j) {
      int slot_next = 0;
      if (j < n_kv) {
        const int st = j % FW_STAGES;
        const int key0 = key0_of(j);
        const int npages = (min(FW_BN, hi - key0) + a.page_size - 1) >> a.page_shift;
        slot_next = lane < npages ? bt[(key0 >> a.page_shift) + lane] * a.page_size : 0;
        if (lane == 0) {
          ok = mbar_wait(&k_empty[st], (j / FW_STAGES & 1) ^ 1, cta_abort, status, ERR_WAIT_EMPTY);
          if (ok) mbar_arrive_expect_tx(&k_full[st], npages * a.page_size * 128 * S::KCH);
        }
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (!ok) break;
        if (lane < npages)
#pragma unroll
          for (int c = 0; c < S::KCH; ++c) {
            uint8_t* dst = sK + st * S::K_BYTES + c * (FW_BN * 128) + lane * a.page_size * 128;
            if (c < a.kchunks) tma_load_3d(dst, &tmK, &k_full[st], c * 64, kvh, slot_next);
            else tma_load_3d(dst, &tmK2, &k_full[st], (c - a.kchunks) * 64, 0, slot_next);
          }
      }
      if (j > 0) {
        const int i = j - 1, st = i % S::VSTAGES;
        const int npages = (min(FW_BN, hi - key0_of(i)) + a.page_size - 1) >> a.page_shift;
        if (lane == 0) {
          ok = mbar_wait(&v_empty[st], (i / S::VSTAGES & 1) ^ 1, cta_abort, status, ERR_WAIT_EMPTY);
          if (ok) mbar_arrive_expect_tx(&v_full[st], npages * a.page_size * 128 * S::VCH);
        }
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (!ok) break;
        if (lane < npages)
#pragma unroll
          for (int c = 0; c < S::VCH; ++c)
            tma_load_3d(sV + st * S::V_BYTES + c * (FW_BN * 128) + lane * a.page_size * 128, &tmV, &v_full[st], c * 64, kvh, slot_k);
      }
      slot_k = slot_next;
    }
  } else if (warp == 1) {
    // -------------------------------------------------------------------- MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc(FW_BM, FW_BN, 1, 1, 0, 0);
      constexpr uint32_t idesc_o = make_idesc(FW_BM, DV, 1, 1, 0, 1);  // B = V read MN-major
      const uint32_t q_addr = smem_u32(sQ), p_addr = smem_u32(sP), x_addr = smem_u32(sX);
      auto issue_s = [&](int j) {
        const uint32_t k_addr = smem_u32(sK + (j % FW_STAGES) * S::K_BYTES);
#pragma unroll
        for (int k = 0; k < DK / 16; ++k) {
          const uint32_t off = (k >> 2) * (FW_BM * 128) + (k & 3) * 32;
          umma_f16(tmem_base + (j & 1) * FW_BN, make_smem_desc(q_addr + off, 16, 1024, UMMA_SWIZZLE_128B),
                   make_smem_desc(k_addr + off, 16, 1024, UMMA_SWIZZLE_128B), idesc_s, k != 0 ? 1u : 0u);
        }
        if (!RULED && S::X_BYTES > 0 && a.rule.slopes != nullptr)
          umma_f16(tmem_base + (j & 1) * FW_BN, make_smem_desc(x_addr, 16, 1024, UMMA_SWIZZLE_128B),
                   make_smem_desc(x_addr + 32, 16, 1024, UMMA_SWIZZLE_128B), idesc_s, 1u);
        umma_commit(&k_empty[j % FW_STAGES]);
        umma_commit(&s_full[j & 1]);
      };
      bool ok = mbar_wait(q_full, 0, cta_abort, status, ERR_WAIT_FULL) && mbar_wait(&k_full[0], 0, cta_abort, status, ERR_WAIT_FULL);
      if (ok) {
        tc_fence_after();
        issue_s(0);
      }
      for (int j = 0; j < n_kv && ok; ++j) {
        if (j + 1 < n_kv) {  // S_{j+1} underneath the softmax of tile j (its buffer was released with p_full of tile j - 1)
          ok = mbar_wait(&k_full[(j + 1) % FW_STAGES], ((j + 1) / FW_STAGES) & 1, cta_abort, status, ERR_WAIT_FULL);
          if (!ok) break;
          tc_fence_after();
          issue_s(j + 1);
        }
        ok = mbar_wait(&v_full[j % S::VSTAGES], (j / S::VSTAGES) & 1, cta_abort, status, ERR_WAIT_FULL);
        if (!ok) break;
        const uint32_t v_addr = smem_u32(sV + (j % S::VSTAGES) * S::V_BYTES);
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          ok = ok && mbar_wait(&p_full[g], j & 1, cta_abort, status, ERR_WAIT_TMEM_EMPTY);
          if (!ok) break;
          tc_fence_after();
#pragma unroll
          for (int k = 0; k < FW_HALF / 16; ++k) {
            const uint64_t da = make_smem_desc(p_addr + g * (FW_BM * 128) + k * 32, 16, 1024, UMMA_SWIZZLE_128B);
            const uint64_t db = make_smem_desc(v_addr + (g * (FW_HALF / 16) + k) * 2048, FW_BN * 128, 1024, UMMA_SWIZZLE_128B);
            umma_f16(tmem_base + 2 * FW_BN + g * DV, da, db, idesc_o, (j != 0 || k != 0) ? 1u : 0u);
          }
          if (g == 1) umma_commit(&v_empty[j % S::VSTAGES]);
          umma_commit(&o_done[g]);
        }
      }
    }
  } else {
    // -------------------------------------------------------------------- softmax + epilogue
    const int quarter = warp & 3, half = warp >= 6;
    const int row = quarter * 32 + lane;  // row of the tile = TMEM lane = token * G + head
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(quarter * 32) << 16);
    const float c_log2 = a.rule.scale * 1.4426950408889634f;
    const int tok = row / G, head = kvh * G + row - tok * G;
    const bool valid = tok < ntok;
    const int pos = p0 + tok;
    const float slope2 = (valid && a.rule.slopes != nullptr) ? a.rule.slopes[head] * 1.4426950408889634f : 0.f;
    const int low = rule_first_key(a.rule, pos);          // first key of this row's window or chunk
    const int low_last = rule_first_key(a.rule, hi - 1);  // ... of the tile's last row
    // RULED: capped score c2 - 2 c2 / (1 + 2^(k x)), see cap_exp2; a distance beyond the table has one bias per row
    const float cap2 = a.rule.softcap * 1.4426950408889634f;
    const float cap_k = RULED && a.rule.softcap > 0.f ? 2.f * c_log2 / a.rule.softcap : 0.f;
    const float* tab = near_table ? reinterpret_cast<const float*>(sX) + (row - tok * G) : a.rule.bias + (valid ? head : 0);
    const int tab_pitch = near_table ? G : a.Hq;
    const float tab_unit = near_table ? 1.f : 1.4426950408889634f;
    const float bias_far = RULED && a.rule.bias != nullptr ? tab[static_cast<size_t>(far) * tab_pitch] * tab_unit : 0.f;
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int j = 0; j < n_kv; ++j) {
      ok = mbar_wait(&s_full[j & 1], (j >> 1) & 1, cta_abort, status, ERR_WAIT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const uint32_t s_addr = lane_addr + (j & 1) * FW_BN + half * FW_HALF;
      const int tile0 = key0_of(j), key0 = tile0 + half * FW_HALF;  // of the tile, of this group's part
      // every row sees the whole part: no element tests (rows past the tile's tokens never do: their scores are garbage)
      const bool masked = key0 + FW_HALF - 1 > p0 || key0 < low_last || ntok < bq || row >= bq * G;
      // bit i of vis[w]: column 32 w + i is visible: c <= up and (c >= dn or c < kp)
      const int up = valid ? pos - key0 : -1, dn = low - key0, kp = a.rule.keep_first - key0;
      uint32_t vis[FW_HALF / 32];
#pragma unroll
      for (int w = 0; w < FW_HALF / 32; ++w)
        vis[w] = fw_below(up + 1 - 32 * w) & (~fw_below(dn - 32 * w) | fw_below(kp - 32 * w));
      const float rowb = slope2 * static_cast<float>(tile0 - pos);
      float mx = -INFINITY;  // plain: of the raw products, as scale > 0 and rowb is the same for the whole row
      float sv[RULED ? FW_HALF : 1];
      if constexpr (RULED) {
        const bool uniform = a.rule.bias == nullptr || p0 - (key0 + FW_HALF - 1) >= far;
#pragma unroll
        for (int c4 = 0; c4 < FW_HALF / 32; ++c4) {
          uint32_t r[32];
          tmem_ld_32x32(s_addr + c4 * 32, r);
          tmem_ld_wait();
          float* s = sv + c4 * 32;
          if (cap_k > 0.f) {
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              const float e0 = cap_exp2(__uint_as_float(r[i]), cap_k), e1 = cap_exp2(__uint_as_float(r[i + 1]), cap_k);
              const float inv = -2.f * cap2 * fast_rcp(e0 * e1);
              s[i] = fmaf(inv, e1, cap2 + bias_far);
              s[i + 1] = fmaf(inv, e0, cap2 + bias_far);
            }
          } else {
#pragma unroll
            for (int i = 0; i < 32; ++i) s[i] = fmaf(__uint_as_float(r[i]), c_log2, bias_far);
          }
          if (!uniform) {
            const int n0 = pos - key0 - c4 * 32;
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              const int n = min(max(n0 - i, 0), far);
              s[i] += fmaf(tab[static_cast<size_t>(n) * tab_pitch], tab_unit, -bias_far);
            }
          }
          if (masked) {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (!(vis[c4] >> i & 1)) s[i] = -INFINITY;
          }
#pragma unroll
          for (int i = 0; i < 32; ++i) mx = fmaxf(mx, s[i]);
        }
      } else {
  #pragma unroll
        for (int c4 = 0; c4 < FW_HALF / 32; ++c4) {
          uint32_t r[32];
          tmem_ld_32x32(s_addr + c4 * 32, r);
          tmem_ld_wait();
          if (masked) {
  #pragma unroll
            for (int i = 0; i < 32; ++i)
              if (vis[c4] >> i & 1) mx = fmaxf(mx, __uint_as_float(r[i]));
          } else {
  #pragma unroll
            for (int i = 0; i < 32; ++i) mx = fmaxf(mx, __uint_as_float(r[i]));
          }
        }
        mx = fmaf(mx, c_log2, rowb);
      }
      const float m_new = fmaxf(m_run, mx);
      bool raise = false;
      if (j == 0) m_run = m_new;
      else raise = __any_sync(0xffffffffu, m_run == -INFINITY ? m_new > -INFINITY : m_new > m_run + 8.f);
      const float m_use = raise ? m_new : m_run;
      const float m_sub = m_use == -INFINITY ? 0.f : m_use;
      uint32_t pk[FW_HALF / 2];
      float lsum = 0.f;
#pragma unroll
      for (int c4 = 0; c4 < FW_HALF / 32; ++c4) {
        if constexpr (RULED) {
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            const float q0 = fw_exp2(sv[c4 * 32 + i] - m_sub), q1 = fw_exp2(sv[c4 * 32 + i + 1] - m_sub);
            lsum += q0 + q1;
            pk[c4 * 16 + (i >> 1)] = pack_bf16x2(q0, q1);
          }
          continue;
        }
        uint32_t r[32];
        tmem_ld_32x32(s_addr + c4 * 32, r);
        tmem_ld_wait();
        const float off = rowb - m_sub;
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          float q0 = fw_exp2(fmaf(__uint_as_float(r[i]), c_log2, off));
          float q1 = fw_exp2(fmaf(__uint_as_float(r[i + 1]), c_log2, off));
          if (masked) {
            if (!(vis[c4] >> i & 1)) q0 = 0.f;
            if (!(vis[c4] >> (i + 1) & 1)) q1 = 0.f;
          }
          lsum += q0 + q1;
          pk[c4 * 16 + (i >> 1)] = pack_bf16x2(q0, q1);
        }
      }
      if (j > 0) {  // the previous product has finished: P may be overwritten and O corrected
        ok = mbar_wait(&o_done[half], (j - 1) & 1, cta_abort, status, ERR_WAIT_TMEM_FULL);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        if (raise) {
          const float f = m_run == -INFINITY ? 0.f : fw_exp2(m_run - m_use);  // <= 1; nothing summed yet: 0
          l_run *= f;
#pragma unroll
          for (int c4 = 0; c4 < DV / 32; ++c4) {
            uint32_t r[32];
            tmem_ld_32x32(lane_addr + 2 * FW_BN + half * DV + c4 * 32, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * f);
            tmem_st_32x32(lane_addr + 2 * FW_BN + half * DV + c4 * 32, r);
          }
          tmem_st_wait();
          m_run = m_use;
        }
      }
      l_run += lsum;
      {
        uint8_t* prow = sP + half * (FW_BM * 128) + row * 128;
        const int sw = row & 7;
#pragma unroll
        for (int i = 0; i < FW_HALF / 8; ++i)
          *reinterpret_cast<uint4*>(prow + ((i ^ sw) << 4)) =
              make_uint4(pk[4 * i], pk[4 * i + 1], pk[4 * i + 2], pk[4 * i + 3]);
      }
      const int nvalid = hi - key0;  // keys of this part that exist
      if (nvalid < FW_HALF) {
        // Value rows past the end hold whatever the page or an older tile left there, or were never written; their p is 0,
        // but 0 x NaN would poison O. Every thread observes the copy's barrier before it overwrites a row.
        const int st = j % S::VSTAGES;
        ok = mbar_wait(&v_full[st], (j / S::VSTAGES) & 1, cta_abort, status, ERR_WAIT_FULL);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        if (row < FW_HALF && row >= nvalid) {
          uint8_t* vrow = sV + st * S::V_BYTES + (half * FW_HALF + row) * 128;
#pragma unroll
          for (int c = 0; c < S::VCH; ++c)
#pragma unroll
            for (int i = 0; i < 8; ++i) reinterpret_cast<uint4*>(vrow + c * (FW_BN * 128))[i] = make_uint4(0, 0, 0, 0);
        }
      }
      fence_proxy_async();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[half]);
    }
    // ---- epilogue: both groups' O, joined, / l -> bf16 -> staged through shared memory (the P buffer) -> rows of `out`. Each group
    // does half of the columns. The queries are no longer needed: their buffer carries the maxima and sums across.
    constexpr int CH = DV / 8;  // 16-byte chunks per output row
    float2* ml = reinterpret_cast<float2*>(sQ);
    for (int g = 0; g < 2 && ok; ++g) ok = mbar_wait(&o_done[g], (n_kv - 1) & 1, cta_abort, status, ERR_WAIT_TMEM_FULL);
    ok = __all_sync(0xffffffffu, ok);
    if (ok) ml[half * FW_BM + row] = make_float2(m_run, l_run);
    asm volatile("bar.sync 1, 256;" ::: "memory");  // all softmax warps, also when a wait has expired
    if (ok) {
      tc_fence_after();
      const float2 other = ml[(half ^ 1) * FW_BM + row];
      const float m = fmaxf(m_run, other.x);
      const float mine = m_run == -INFINITY ? 0.f : fw_exp2(m_run - m), theirs = other.x == -INFINITY ? 0.f : fw_exp2(other.x - m);
      float l = l_run * mine + other.y * theirs;
      if (valid && a.rule.sinks != nullptr) l += fw_exp2(fmaf(a.rule.sinks[head], 1.4426950408889634f, -m));
      float inv = l > 0.f ? a.rule.out_scale / l : 0.f;
      const __nv_bfloat16* gate = nullptr;  // of this row; one number for the head is part of inv
      if (valid && a.rule.gate != nullptr) {
        gate = reinterpret_cast<const __nv_bfloat16*>(a.rule.gate) + static_cast<size_t>(row0 + tok) * a.rule.gate_pitch +
               static_cast<size_t>(head) * a.rule.gate_width;
        if (a.rule.gate_width == 1) {
          inv *= sigmoid_f(__bfloat162float(*gate));
          gate = nullptr;
        }
      }
      const float f0 = inv * (half == 0 ? mine : theirs), f1 = inv * (half == 0 ? theirs : mine);
      if constexpr (PAIR) {
        float x[DV / 2], ss = 0.f;  // columns half * DV / 2 ...
#pragma unroll
        for (int c = 0; c < DV / 64; ++c) {
          uint32_t r[32], r1[32];
          tmem_ld_32x32(lane_addr + 2 * FW_BN + half * (DV / 2) + c * 32, r);
          tmem_ld_32x32(lane_addr + 2 * FW_BN + DV + half * (DV / 2) + c * 32, r1);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float o = fmaf(__uint_as_float(r[i]), f0, __uint_as_float(r1[i]) * f1);
            const float y = fmaf(-a.rule.pair[0], __shfl_xor_sync(0xffffffffu, o, 1), o);  // (of even rows)
            x[c * 32 + i] = y;
            ss = fmaf(y, y, ss);
          }
        }
        float* sums = reinterpret_cast<float*>(ml + 2 * FW_BM);
        sums[half * FW_BM + row] = ss;
        asm volatile("bar.sync 2, 256;" ::: "memory");
        const float r = a.rule.pair_gain / sqrtf((ss + sums[(half ^ 1) * FW_BM + row]) / a.dv + a.rule.pair_eps);
        if (!(row & 1)) {
          const int rr = row >> 1;
          uint8_t* orow = sP + rr * (DV * 2);
#pragma unroll
          for (int i = 0; i < DV / 16; ++i) {
            const int ch = half * (DV / 16) + i;
            *reinterpret_cast<uint4*>(orow + ((ch ^ (rr & (CH - 1))) << 4)) =
                make_uint4(pack_bf16x2(x[8 * i] * r, x[8 * i + 1] * r), pack_bf16x2(x[8 * i + 2] * r, x[8 * i + 3] * r),
                           pack_bf16x2(x[8 * i + 4] * r, x[8 * i + 5] * r), pack_bf16x2(x[8 * i + 6] * r, x[8 * i + 7] * r));
          }
        }
      } else {
      uint8_t* orow = sP + row * (DV * 2);
#pragma unroll
      for (int c = 0; c < DV / 64; ++c) {
        const int c4 = half * (DV / 64) + c;
        uint32_t r[32], r1[32];
        tmem_ld_32x32(lane_addr + 2 * FW_BN + c4 * 32, r);
        tmem_ld_32x32(lane_addr + 2 * FW_BN + DV + c4 * 32, r1);
        tmem_ld_wait();
        // a group that has seen nothing has multiplied by zeros only: its O is 0
#pragma unroll
        for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(fmaf(__uint_as_float(r[i]), f0, __uint_as_float(r1[i]) * f1));
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int ch = c4 * 4 + i;
          if (gate != nullptr && ch * 8 < a.dv) {
            const uint4 g = *reinterpret_cast<const uint4*>(gate + ch * 8);
            const uint32_t gs[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              const float2 z = unpack_bf16x2(gs[k]);
              r[8 * i + 2 * k] = __float_as_uint(__uint_as_float(r[8 * i + 2 * k]) * sigmoid_f(z.x));
              r[8 * i + 2 * k + 1] = __float_as_uint(__uint_as_float(r[8 * i + 2 * k + 1]) * sigmoid_f(z.y));
            }
          }
          *reinterpret_cast<uint4*>(orow + ((ch ^ (row & (CH - 1))) << 4)) =
              make_uint4(pack_bf16x2(__uint_as_float(r[8 * i]), __uint_as_float(r[8 * i + 1])),
                         pack_bf16x2(__uint_as_float(r[8 * i + 2]), __uint_as_float(r[8 * i + 3])),
                         pack_bf16x2(__uint_as_float(r[8 * i + 4]), __uint_as_float(r[8 * i + 5])),
                         pack_bf16x2(__uint_as_float(r[8 * i + 6]), __uint_as_float(r[8 * i + 7])));
        }
      }
      }
    } else if constexpr (PAIR) {
      asm volatile("bar.sync 2, 256;" ::: "memory");  // the exchange of sums, also when a wait has expired
    }
    asm volatile("bar.sync 1, 256;" ::: "memory");
    if (ok && *cta_abort == 0) {
      const int G = PAIR ? a.G / 2 : a.G;  // output heads of this kv head
      const int t = threadIdx.x - 64, ch_used = a.dv / 8, rows_used = ntok * G;
      for (int idx = t; idx < rows_used * ch_used; idx += 256) {
        const int rr = idx / ch_used, ch = idx - rr * ch_used;
        const int tk = rr / G, hd = kvh * G + rr - tk * G;
        *reinterpret_cast<uint4*>(a.out + static_cast<size_t>(row0 + tk) * a.out_stride + hd * a.dv + ch * 8) =
            *reinterpret_cast<const uint4*>(sP + rr * (DV * 2) + ((ch ^ (rr & (CH - 1))) << 4));
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
  if (warp == 1) tmem_dealloc(tmem_base, S::TMEM_COLS);
}

// [rows, heads, width] bf16 with a free pitch between rows (and between heads: head_pitch, 0 = width); box = [rows, box_heads,
// 64]. Columns past `width` read as zero, which pads a head to the tile's width.
static CUtensorMap fw_map(const void* base, uint64_t width, uint64_t heads, uint64_t rows, uint64_t row_pitch, uint32_t box_heads,
                          uint32_t box_rows, uint64_t head_pitch = 0) {
  return make_tmap_3d(base, width, heads, rows, head_pitch ? head_pitch : width, row_pitch, 64, box_heads, box_rows);
}

struct FwMaps {
  CUtensorMap q, k, v, q2, k2;
};

template <int DK, int DV>
static int launch_flash_window(dim3 grid, const FwMaps& m, const FwArgs& a, cudaStream_t s) {
  constexpr int bytes = FwSmem<DK, DV>::TOTAL;
  const bool ruled = a.rule.softcap > 0.f || a.rule.bias != nullptr;
  auto kern = ruled ? flash_window_kernel<DK, DV, FW_RULED> : flash_window_kernel<DK, DV, FW_PLAIN>;
  if (a.rule.pair != nullptr) {
    if constexpr (DK > 128) return -1;
    else kern = flash_window_kernel<DK, DV, FW_PAIR>;
  }
  if (cudaError_t e = ensure_dynamic_smem(reinterpret_cast<const void*>(kern), bytes); e != cudaSuccess) return (int)e;
  return (int)launch_pdl(kern, grid, dim3(FW_THREADS), bytes, s, m.q, m.k, m.v, m.q2, m.k2, a);
}

// What both entry points check: groups, page size, alignment of everything the kernel moves in 16-byte pieces.
static bool fw_takes(const AttnRule& r, int G, int DV, int page_size, int* shift, long q_stride, long out_stride, uintptr_t pointers) {
  if (G > FW_BM || DV <= 0 || DV > 128 || DV % 8 || !rule_pairs_ok(&r, G)) return false;
  if (r.slopes != nullptr && (r.softcap > 0.f || r.bias != nullptr)) return false;
  *shift = 0;
  while ((1 << *shift) < page_size) ++*shift;
  if ((1 << *shift) != page_size || page_size < 16 || page_size > 128) return false;
  if (r.gate != nullptr && r.gate_width > 1 && ((reinterpret_cast<uintptr_t>(r.gate) & 15) || r.gate_pitch % 8)) return false;
  return (pointers & 15) == 0 && q_stride % 8 == 0 && out_stride % 8 == 0;
}

}  // namespace sb

// q [T, Hq, D] bf16 (heads adjacent, row pitch q_stride), caches [num_slots, Hkv, D] and [num_slots, Hkv, DV] contiguous;
// block_table rows of max_pages ints; tiles: ntiles x int4 as described above with at most 128 / (Hq / Hkv) tokens each;
// out [T, Hq * DV] (pairs: half as many heads) with row pitch out_stride; attn_rule: AttnRule. D, DV multiples of 8 up to 128.
// Returns 0, a cudaError_t value, or -1 when the shape or an alignment is outside what the kernel takes.
extern "C" int sb_flash_window(const void* q, const void* k_cache, const void* v_cache, const int* block_table, const int* tiles,
                               void* out, int ntiles, int T, int Hq, int Hkv, int D, int DV, int page_size, int max_pages,
                               int num_slots, long q_stride, long out_stride, const void* attn_rule, int* status, cudaStream_t s) {
  if (ntiles <= 0 || T <= 0) return 0;
  const sb::AttnRule* rule = (const sb::AttnRule*)attn_rule;
  if (Hkv <= 0 || Hq % Hkv != 0 || !rule_ok(rule)) return (int)cudaErrorInvalidValue;
  const int G = Hq / Hkv;
  int shift = 0;
  if (D <= 0 || D > 128 || D % 8 ||
      !sb::fw_takes(*rule, G, DV, page_size, &shift, q_stride, out_stride,
                    reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) |
                        reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(tiles)))
    return -1;
  try {
    sb::FwMaps m;
    m.q = m.q2 = sb::fw_map(q, D, Hq, T, q_stride, G, sb::FW_BM / G);
    m.k = m.k2 = sb::fw_map(k_cache, D, Hkv, num_slots, long(Hkv) * D, 1, page_size);
    m.v = sb::fw_map(v_cache, DV, Hkv, num_slots, long(Hkv) * DV, 1, page_size);
    const sb::FwArgs a{block_table, reinterpret_cast<const int4*>(tiles), (__nv_bfloat16*)out, Hq, Hkv, G, DV, page_size, shift, max_pages,
                       D <= 64 ? 1 : 2, out_stride, status, *rule};
    const dim3 grid(ntiles, Hkv);
    if (D <= 64 && DV <= 64) return sb::launch_flash_window<64, 64>(grid, m, a, s);
    if (D <= 64) return sb::launch_flash_window<64, 128>(grid, m, a, s);
    if (DV <= 64) return sb::launch_flash_window<128, 64>(grid, m, a, s);
    return sb::launch_flash_window<128, 128>(grid, m, a, s);
  } catch (const std::exception& e) {
    sb::set_last_error(e.what());
    return (int)cudaErrorInvalidValue;
  }
}

// Latent attention with expanded keys and values, one head per tile: q [T, H, D + R] (row pitch q_stride), of which the first D
// coordinates meet k [num_slots, H, D] and the last R meet `shared` [num_slots, R], the same for every head; v [num_slots, H, DV].
// Row pitches k_pitch, shared_pitch, v_pitch in elements. The rest as above. D, R, DV multiples of 8; R up to 64, D and DV up to 128.
extern "C" int sb_flash_latent(const void* q, const void* k, const void* shared, const void* v, const int* block_table, const int* tiles,
                               void* out, int ntiles, int T, int H, int D, int R, int DV, int page_size, int max_pages,
                               int num_slots, long q_stride, long k_pitch, long shared_pitch, long v_pitch, long out_stride,
                               const void* attn_rule, int* status, cudaStream_t s) {
  if (ntiles <= 0 || T <= 0) return 0;
  const sb::AttnRule* rule = (const sb::AttnRule*)attn_rule;
  if (H <= 0 || !rule_ok(rule)) return (int)cudaErrorInvalidValue;
  int shift = 0;
  if (D <= 0 || D > 128 || D % 8 || R <= 0 || R > 64 || R % 8 || rule->slopes != nullptr || rule->softcap > 0.f || rule->bias != nullptr ||
      k_pitch % 8 || shared_pitch % 8 || v_pitch % 8 ||
      !sb::fw_takes(*rule, 1, DV, page_size, &shift, q_stride, out_stride,
                    reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(shared) |
                        reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(tiles)))
    return -1;
  try {
    using bf16 = __nv_bfloat16;
    sb::FwMaps m;
    m.q = sb::fw_map(q, D, H, T, q_stride, 1, sb::FW_BM, D + R);
    m.q2 = sb::fw_map((const bf16*)q + D, R, H, T, q_stride, 1, sb::FW_BM, D + R);
    m.k = sb::fw_map(k, D, H, num_slots, k_pitch, 1, page_size);
    m.k2 = sb::fw_map(shared, R, 1, num_slots, shared_pitch, 1, page_size);
    m.v = sb::fw_map(v, DV, H, num_slots, v_pitch, 1, page_size);
    const sb::FwArgs a{block_table, reinterpret_cast<const int4*>(tiles), (bf16*)out, H, H, 1, DV, page_size, shift, max_pages,
                       D <= 64 ? 1 : 2, out_stride, status, *rule};
    const dim3 grid(ntiles, H);
    if (D <= 64 && DV <= 64) return sb::launch_flash_window<128, 64>(grid, m, a, s);
    if (D <= 64) return sb::launch_flash_window<128, 128>(grid, m, a, s);
    if (DV <= 64) return sb::launch_flash_window<192, 64>(grid, m, a, s);
    return sb::launch_flash_window<192, 128>(grid, m, a, s);
  } catch (const std::exception& e) {
    sb::set_last_error(e.what());
    return (int)cudaErrorInvalidValue;
  }
}
