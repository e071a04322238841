// Windowed attention of prompt rows over the paged KV cache, on the 5th-gen tensor cores (sm_100a). Sister of
// flash_fwd_sm100.cu (same warp roles, same softmax scheme) for layers whose queries see a sliding window plus the first
// tokens of the sequence and whose scores carry a linear distance penalty:
//
//     row at position i sees key j   iff   j <= i  and  (i - j < window  or  j < keep_first)
//     score = scale * q.k - slope[head] * (i - j)                                     (slopes null: no penalty)
// sinks: score of an extra softmax column that has no value, per head (null: none); it joins the sum once, at the end. The
// output is multiplied by out_scale.
//
// Two things differ in structure. Keys and values come straight from the cache pages (one TMA box per page and 64-wide
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
#include "common.cuh"

namespace sb {

constexpr int FW_BM = 128, FW_BN = 128;
constexpr int FW_THREADS = 192;  // TMA warp, MMA warp, 4 softmax warps
constexpr int FW_STAGES = 2;

template <int DK, int DV>
struct FwSmem {
  static constexpr int KCH = DK / 64, VCH = DV / 64;
  static constexpr int Q_BYTES = FW_BM * 128 * KCH;
  static constexpr int K_BYTES = FW_BN * 128 * KCH;
  static constexpr int V_BYTES = FW_BN * 128 * VCH;
  static constexpr int P_BYTES = FW_BM * FW_BN * 2;
  static constexpr int X_BYTES = FW_BM * 128;  // extra columns: k-step 0 of row r = query row r's, k-step 1 = key column r's
  static constexpr int TOTAL = Q_BYTES + FW_STAGES * (K_BYTES + V_BYTES) + P_BYTES + X_BYTES + 256 + 1024;  // + barriers, alignment
  static constexpr int TMEM_COLS = 512;  // S0 @0, S1 @128, O @256
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
  const float *slopes, *sinks;
  __nv_bfloat16* out;
  int Hkv, G, dv, page_size, page_shift, max_pages;
  long out_stride;
  float scale, out_scale;
  int window, keep_first;
  int* status;
};

template <int DK, int DV>
__global__ void __launch_bounds__(FW_THREADS, 1)
flash_window_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                    const __grid_constant__ CUtensorMap tmV, const __grid_constant__ FwArgs a) {
  using S = FwSmem<DK, DV>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + S::Q_BYTES;
  uint8_t* sV = sK + FW_STAGES * S::K_BYTES;
  uint8_t* sP = sV + FW_STAGES * S::V_BYTES;
  uint8_t* sX = sP + S::P_BYTES;
  uint64_t* q_full = reinterpret_cast<uint64_t*>(sX + S::X_BYTES);
  uint64_t* k_full = q_full + 1;
  uint64_t* k_empty = k_full + FW_STAGES;
  uint64_t* v_full = k_empty + FW_STAGES;
  uint64_t* v_empty = v_full + FW_STAGES;
  uint64_t* s_full = v_empty + FW_STAGES;  // [2]
  uint64_t* p_full = s_full + 2;
  uint64_t* o_done = p_full + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 1);
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
    mbar_init(p_full, 4);  // one arrival per softmax warp
    mbar_init(o_done, 1);
    *cta_abort = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, S::TMEM_COLS);
    tmem_relinquish();
  }
  pdl_wait();
  pdl_launch_dependents();
  if (a.slopes != nullptr && warp >= 2) {
    const int r = threadIdx.x - 64;
    const float f = r < bq * G ? a.slopes[kvh * G + r % G] / a.scale : 0.f;
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
  const int lo = a.window > p0 ? 0 : p0 - a.window + 1;             // first key of the first row's window
  int base = (lo >> a.page_shift) << a.page_shift;                  // windowed tiles start at a page
  const int n_keep = min((min(a.keep_first, hi) + FW_BN - 1) / FW_BN, (base + FW_BN - 1) / FW_BN);
  base = max(base, n_keep * FW_BN);
  const int n_kv = n_keep + (hi > base ? (hi - base + FW_BN - 1) / FW_BN : 0);
  auto key0_of = [&](int j) { return j < n_keep ? j * FW_BN : base + (j - n_keep) * FW_BN; };

  if (warp == 0) {
    // -------------------------------------------------------------------- TMA producer (lane p: page p of the tile)
    if (lane == 0) {
      mbar_arrive_expect_tx(q_full, bq * G * 128 * S::KCH);
#pragma unroll
      for (int c = 0; c < S::KCH; ++c) tma_load_3d(sQ + c * (FW_BM * 128), &tmQ, q_full, c * 64, kvh * G, row0);
    }
    bool ok = true;
    for (int j = 0; j < n_kv && ok; ++j) {
      const int st = j % FW_STAGES;
      const uint32_t par = (j / FW_STAGES) & 1;
      const int key0 = key0_of(j);
      const int npages = (min(FW_BN, hi - key0) + a.page_size - 1) >> a.page_shift;
      const int slot0 = lane < npages ? bt[(key0 >> a.page_shift) + lane] * a.page_size : 0;
      if (lane == 0) {
        ok = mbar_wait(&k_empty[st], par ^ 1, cta_abort, status, ERR_WAIT_EMPTY);
        if (ok) mbar_arrive_expect_tx(&k_full[st], npages * a.page_size * 128 * S::KCH);
      }
      ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
      if (!ok) break;
      if (lane < npages)
#pragma unroll
        for (int c = 0; c < S::KCH; ++c)
          tma_load_3d(sK + st * S::K_BYTES + c * (FW_BN * 128) + lane * a.page_size * 128, &tmK, &k_full[st], c * 64, kvh, slot0);
      if (lane == 0) {
        ok = mbar_wait(&v_empty[st], par ^ 1, cta_abort, status, ERR_WAIT_EMPTY);
        if (ok) mbar_arrive_expect_tx(&v_full[st], npages * a.page_size * 128 * S::VCH);
      }
      ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
      if (!ok) break;
      if (lane < npages)
#pragma unroll
        for (int c = 0; c < S::VCH; ++c)
          tma_load_3d(sV + st * S::V_BYTES + c * (FW_BN * 128) + lane * a.page_size * 128, &tmV, &v_full[st], c * 64, kvh, slot0);
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
        if (a.slopes != nullptr)
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
        ok = mbar_wait(p_full, j & 1, cta_abort, status, ERR_WAIT_TMEM_EMPTY) &&
             mbar_wait(&v_full[j % FW_STAGES], (j / FW_STAGES) & 1, cta_abort, status, ERR_WAIT_FULL);
        if (!ok) break;
        tc_fence_after();
        const uint32_t v_addr = smem_u32(sV + (j % FW_STAGES) * S::V_BYTES);
#pragma unroll
        for (int k = 0; k < FW_BN / 16; ++k) {
          const uint64_t da = make_smem_desc(p_addr + (k >> 2) * (FW_BM * 128) + (k & 3) * 32, 16, 1024, UMMA_SWIZZLE_128B);
          const uint64_t db = make_smem_desc(v_addr + k * 2048, FW_BN * 128, 1024, UMMA_SWIZZLE_128B);
          umma_f16(tmem_base + 2 * FW_BN, da, db, idesc_o, (j != 0 || k != 0) ? 1u : 0u);
        }
        umma_commit(&v_empty[j % FW_STAGES]);
        umma_commit(o_done);
      }
    }
  } else {
    // -------------------------------------------------------------------- softmax + epilogue
    const int quarter = warp & 3;
    const int row = quarter * 32 + lane;  // row of the tile = TMEM lane = token * G + head
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(quarter * 32) << 16);
    const float c_log2 = a.scale * 1.4426950408889634f;
    const int tok = row / G, head = kvh * G + row - tok * G;
    const bool valid = tok < ntok;
    const int pos = p0 + tok;
    const float slope2 = (valid && a.slopes != nullptr) ? a.slopes[head] * 1.4426950408889634f : 0.f;
    const int low = a.window > pos ? 0 : pos - a.window + 1;            // first key of this row's window
    const int low_last = a.window > hi - 1 ? 0 : hi - a.window;         // ... of the tile's last row
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int j = 0; j < n_kv; ++j) {
      ok = mbar_wait(&s_full[j & 1], (j >> 1) & 1, cta_abort, status, ERR_WAIT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const uint32_t s_addr = lane_addr + (j & 1) * FW_BN;
      const int key0 = key0_of(j);
      // every row sees the whole tile: no element tests (rows past the tile's tokens never do: their scores are garbage)
      const bool masked = key0 + FW_BN - 1 > p0 || key0 < low_last || ntok < bq || row >= bq * G;
      // bit i of vis[w]: column 32 w + i is visible: c <= up and (c >= dn or c < kp)
      const int up = valid ? pos - key0 : -1, dn = low - key0, kp = a.keep_first - key0;
      uint32_t vis[FW_BN / 32];
#pragma unroll
      for (int w = 0; w < FW_BN / 32; ++w)
        vis[w] = fw_below(up + 1 - 32 * w) & (~fw_below(dn - 32 * w) | fw_below(kp - 32 * w));
      const float rowb = slope2 * static_cast<float>(key0 - pos);
      float mx = -INFINITY;  // of the raw products: scale > 0 and rowb is the same for the whole row
#pragma unroll
      for (int c4 = 0; c4 < FW_BN / 32; ++c4) {
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
      const float m_new = fmaxf(m_run, mx);
      bool raise = false;
      if (j == 0) m_run = m_new;
      else raise = __any_sync(0xffffffffu, m_run == -INFINITY ? m_new > -INFINITY : m_new > m_run + 8.f);
      const float m_use = raise ? m_new : m_run;
      const float m_sub = m_use == -INFINITY ? 0.f : m_use;
      uint32_t pk[FW_BN / 2];
      float lsum = 0.f;
#pragma unroll
      for (int c4 = 0; c4 < FW_BN / 32; ++c4) {
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
        ok = mbar_wait(o_done, (j - 1) & 1, cta_abort, status, ERR_WAIT_TMEM_FULL);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        if (raise) {
          const float f = m_run == -INFINITY ? 0.f : fw_exp2(m_run - m_use);  // <= 1; nothing summed yet: 0
          l_run *= f;
#pragma unroll
          for (int c4 = 0; c4 < DV / 32; ++c4) {
            uint32_t r[32];
            tmem_ld_32x32(lane_addr + 2 * FW_BN + c4 * 32, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * f);
            tmem_st_32x32(lane_addr + 2 * FW_BN + c4 * 32, r);
          }
          tmem_st_wait();
          m_run = m_use;
        }
      }
      l_run += lsum;
      {
        uint8_t* prow = sP + row * 128;
        const int sw = row & 7;
#pragma unroll
        for (int i = 0; i < FW_BN / 8; ++i)
          *reinterpret_cast<uint4*>(prow + (i >> 3) * (FW_BM * 128) + (((i & 7) ^ sw) << 4)) =
              make_uint4(pk[4 * i], pk[4 * i + 1], pk[4 * i + 2], pk[4 * i + 3]);
      }
      const int nvalid = hi - key0;  // keys of this tile that exist
      if (nvalid < FW_BN) {
        // Value rows past the end hold whatever the page or an older tile left there, or were never written; their p is 0,
        // but 0 x NaN would poison O. Every thread observes the copy's barrier before it overwrites a row.
        const int st = j % FW_STAGES;
        ok = mbar_wait(&v_full[st], (j / FW_STAGES) & 1, cta_abort, status, ERR_WAIT_FULL);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        if (row >= nvalid) {
          uint8_t* vrow = sV + st * S::V_BYTES + row * 128;
#pragma unroll
          for (int c = 0; c < S::VCH; ++c)
#pragma unroll
            for (int i = 0; i < 8; ++i) reinterpret_cast<uint4*>(vrow + c * (FW_BN * 128))[i] = make_uint4(0, 0, 0, 0);
        }
      }
      fence_proxy_async();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    // ---- epilogue: O / l -> bf16 -> staged through shared memory (the P buffer) -> rows of `out`
    constexpr int CH = DV / 8;  // 16-byte chunks per output row
    if (ok) {
      ok = mbar_wait(o_done, (n_kv - 1) & 1, cta_abort, status, ERR_WAIT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
    }
    if (ok) {
      tc_fence_after();
      if (valid && a.sinks != nullptr) l_run += fw_exp2(fmaf(a.sinks[head], 1.4426950408889634f, -m_run));
      const float inv = l_run > 0.f ? a.out_scale / l_run : 0.f;
      uint8_t* orow = sP + row * (DV * 2);
#pragma unroll
      for (int c4 = 0; c4 < DV / 32; ++c4) {
        uint32_t r[32];
        tmem_ld_32x32(lane_addr + 2 * FW_BN + c4 * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int ch = c4 * 4 + i;
          *reinterpret_cast<uint4*>(orow + ((ch ^ (row & (CH - 1))) << 4)) =
              make_uint4(pack_bf16x2(__uint_as_float(r[8 * i]) * inv, __uint_as_float(r[8 * i + 1]) * inv),
                         pack_bf16x2(__uint_as_float(r[8 * i + 2]) * inv, __uint_as_float(r[8 * i + 3]) * inv),
                         pack_bf16x2(__uint_as_float(r[8 * i + 4]) * inv, __uint_as_float(r[8 * i + 5]) * inv),
                         pack_bf16x2(__uint_as_float(r[8 * i + 6]) * inv, __uint_as_float(r[8 * i + 7]) * inv));
        }
      }
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");  // the four softmax warps, also when a wait has expired
    if (ok && *cta_abort == 0) {
      const int t = threadIdx.x - 64, ch_used = a.dv / 8, rows_used = ntok * G;
      for (int idx = t; idx < rows_used * ch_used; idx += 128) {
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

// [outer, heads, width] bf16 with a free pitch between outer rows; box = [rows, box_heads, 64]. Columns past `width` read as
// zero, which pads a head to the tile's width.
static CUtensorMap fw_map(const void* base, uint64_t width, uint64_t heads, uint64_t rows, uint64_t row_pitch, uint32_t box_heads,
                          uint32_t box_rows) {
  CUtensorMap m;
  cuuint64_t dims[3] = {width, heads, rows};
  cuuint64_t strides[2] = {width * 2, row_pitch * 2};
  cuuint32_t box[3] = {64, box_heads, box_rows};
  cuuint32_t estr[3] = {1, 1, 1};
  static thread_local bool ctx_bound = false;  // the encoder needs the primary context current on this thread
  if (!ctx_bound) {
    int dev = 0;
    if (cudaGetDevice(&dev) == cudaSuccess && cudaSetDevice(dev) == cudaSuccess) ctx_bound = true;
  }
  CUresult r = get_encode_tiled()(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
                                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS)
    throw std::runtime_error("cuTensorMapEncodeTiled (windowed attention) failed: " + std::to_string(int(r)) + " width=" +
                             std::to_string(width) + " heads=" + std::to_string(heads) + " rows=" + std::to_string(rows));
  return m;
}

template <int DK, int DV>
static int launch_flash_window(dim3 grid, const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& v, const FwArgs& a,
                               cudaStream_t s) {
  auto kern = flash_window_kernel<DK, DV>;
  if (cudaError_t e = ensure_dynamic_smem(reinterpret_cast<const void*>(kern), FwSmem<DK, DV>::TOTAL); e != cudaSuccess) return (int)e;
  return (int)launch_pdl(kern, grid, dim3(FW_THREADS), FwSmem<DK, DV>::TOTAL, s, q, k, v, a);
}

}  // namespace sb

// q [T, Hq, D] bf16 (heads adjacent, row pitch q_stride), caches [num_slots, Hkv, D] and [num_slots, Hkv, DV] contiguous;
// block_table rows of max_pages ints; tiles: ntiles x int4 as described above with at most 128 / (Hq / Hkv) tokens each;
// slopes [Hq] fp32 or null; out [T, Hq * DV] with row pitch out_stride. D, DV multiples of 8 up to 128.
// Returns 0, a cudaError_t value, or -1 when the shape or an alignment is outside what the kernel takes.
extern "C" int sb_flash_window(const void* q, const void* k_cache, const void* v_cache, const int* block_table, const int* tiles,
                               const float* slopes, const float* sinks, void* out, int ntiles, int T, int Hq, int Hkv, int D, int DV, int page_size,
                               int max_pages, int num_slots, long q_stride, long out_stride, float scale, float out_scale,
                               int window, int keep_first, int* status, cudaStream_t s) {
  if (ntiles <= 0 || T <= 0) return 0;
  if (Hkv <= 0 || Hq % Hkv != 0 || window < 1 || keep_first < 0) return (int)cudaErrorInvalidValue;
  const int G = Hq / Hkv;
  if (!(scale > 0.f)) return -1;
  if (G > sb::FW_BM || D <= 0 || DV <= 0 || D > 128 || DV > 128 || D % 8 || DV % 8) return -1;
  int shift = 0;
  while ((1 << shift) < page_size) ++shift;
  if ((1 << shift) != page_size || page_size < 16 || page_size > 128) return -1;
  if (((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) |
        reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(tiles)) & 15) || q_stride % 8 || out_stride % 8)
    return -1;
  try {
    const CUtensorMap tq = sb::fw_map(q, D, Hq, T, q_stride, G, sb::FW_BM / G);
    const CUtensorMap tk = sb::fw_map(k_cache, D, Hkv, num_slots, long(Hkv) * D, 1, page_size);
    const CUtensorMap tv = sb::fw_map(v_cache, DV, Hkv, num_slots, long(Hkv) * DV, 1, page_size);
    const sb::FwArgs a{block_table, reinterpret_cast<const int4*>(tiles), slopes, sinks, (__nv_bfloat16*)out, Hkv, G, DV, page_size, shift,
                       max_pages, out_stride, scale, out_scale, window, keep_first, status};
    const dim3 grid(ntiles, Hkv);
    if (D <= 64 && DV <= 64) return sb::launch_flash_window<64, 64>(grid, tq, tk, tv, a, s);
    if (D <= 64) return sb::launch_flash_window<64, 128>(grid, tq, tk, tv, a, s);
    if (DV <= 64) return sb::launch_flash_window<128, 64>(grid, tq, tk, tv, a, s);
    return sb::launch_flash_window<128, 128>(grid, tq, tk, tv, a, s);
  } catch (const std::exception& e) {
    sb::set_last_error(e.what());
    return (int)cudaErrorInvalidValue;
  }
}
