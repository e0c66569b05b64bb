// Paged causal attention over shared key rows, prompt portions of bfloat16 on the tcgen05 tensor cores: every query head
// of a token reads the same key row (all kv heads' keys side by side, padded to panels of 64 values: up to 8 panels), head
// h has the values of its own kv head.  This is what attention with mixed ("talking") heads comes to once the mixture
// has moved to the queries (talking_heads.cu).
//
// The scheme is that of attention_tcgen05.cu: one CTA per (tile of 128 rows, kv head, sequence), a row a (token, head of
// the kv head's group) pair; key tiles of 64 keys (128 with more
// than four panels) at absolute positions; S = Q K^T and P V as tcgen05.mma with
// accumulators in tensor memory; eight softmax warps, two threads a row; the kept first keys' tiles walked ahead of the
// recent ones.  What differs: the contraction of S is up to eight panels long, so the keys come through a ring of single
// panels (a tile's keys x 64 values), each handed back as soon as its four products are done; and several producer warps share
// out a tile's pages (a box costs its warp some 140 cycles, and a tile has up to 8 panels x 8 pages of them).
// Up to four panels two CTAs share an SM, with more one fills it.
// Decoded tokens, and what the tcgen05 form does not take: the mma.sync kernel of latent_attention_mma.cuh, keys in splits
// where there are few rows.
// Every mbarrier wait is bounded (bit 16 of the error word, then wind-down).  No cluster, no multicast.
#include "attention_tcgen05.cuh"
#include "latent_attention_mma.cuh"

#define SK_BM 128
template <bool BIG> constexpr int sk_producers() { return BIG ? 4 : 2; }
template <bool BIG> constexpr int sk_threads() { return 32 * (sk_producers<BIG>() + 9); }
template <bool BIG> constexpr int sk_keys() { return BIG ? 128 : 64; }           // keys a tile
template <bool BIG> constexpr int sk_panel() { return sk_keys<BIG>() * 128; }     // bytes of a K or V panel: a tile's keys x 64 values
template <int DV, bool BIG> constexpr int sk_vstages() { return 128 / DV; }
#define SK_KSTAGES 4
template <int DV, bool BIG> constexpr int sk_smem(int panels) {
  return panels * 16384 + SK_KSTAGES * sk_panel<BIG>() + sk_vstages<DV, BIG>() * (DV / 64) * sk_panel<BIG>() + 512;
}

template <int DV, bool BIG>
__global__ void __launch_bounds__(sk_threads<BIG>(), BIG ? 1 : 2)
shared_key_tcgen05_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                          const __grid_constant__ CUtensorMap map_v, bf16* out, const int* block_table, int max_blocks,
                          const int* q_start, const int* seq_lens, int seq_begin, int seq_end, int nq, int nkv, int panels,
                          int dv, int page_size, int num_pages, int window, int keep_first, float scale_log2, int* err) {
  constexpr int NP = sk_producers<BIG>(), KST = SK_KSTAGES, VST = sk_vstages<DV, BIG>(), DP = DV / 64;
  constexpr int SK_BN = sk_keys<BIG>(), SK_PANEL = sk_panel<BIG>(), TMEM = BIG ? 512 : 256;
  constexpr int VSTAGE = DP * SK_PANEL;
  extern __shared__ __align__(1024) unsigned char sk_raw[];
  if (tg_smem(sk_raw) & 1023u) {                  // the swizzled tiles need 1024-byte alignment
    if (threadIdx.x == 0) atomicOr(err, 32);
    return;
  }
  unsigned char* sQ = sk_raw;                     // panels x [128 rows][64 values], 128B swizzle
  unsigned char* sK = sQ + panels * 16384;        // KST x [BN keys][64 values]
  unsigned char* sV = sK + KST * SK_PANEL;        // VST x DP x [BN keys][64 values]
  unsigned long long* bars = (unsigned long long*)(sV + VST * VSTAGE);
  unsigned long long* q_full = bars;              // TMA -> MMA
  unsigned long long* k_full = bars + 1;          // [KST] TMA (all producers) -> MMA
  unsigned long long* k_empty = k_full + KST;     // [KST] MMA -> TMA
  unsigned long long* v_full = k_empty + KST;     // [VST] TMA -> MMA, softmax (last tile)
  unsigned long long* v_empty = v_full + VST;     // [VST] MMA -> TMA
  unsigned long long* s_full = v_empty + VST;     // MMA -> softmax
  unsigned long long* p_full = s_full + 1;        // softmax (8 warps) -> MMA
  unsigned long long* pv_full = s_full + 2;       // MMA -> softmax
  unsigned long long* s_free = s_full + 3;        // softmax (8 warps) -> MMA
  unsigned long long* xbar = s_full + 4;          // [4] the two warps of a row quarter, one another
  unsigned* tmem_slot = (unsigned*)(xbar + 4);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = nq / nkv, bq = SK_BM / g;
  const int kvh = blockIdx.x % nkv;
  int s = -1, tile = 0;
  {
    int left = blockIdx.x / nkv;
    for (int i = seq_begin; i < seq_end; ++i) {
      const int n = (q_start[i + 1] - q_start[i] + bq - 1) / bq;
      if (left < n) { s = i; tile = n - 1 - left; break; }
      left -= n;
    }
  }
  if (s < 0) return;
  const int qs = q_start[s], qlen = q_start[s + 1] - qs;
  const int pos0 = seq_lens[s] - qlen;
  const int t0 = tile * bq;
  const int ntok = min(bq, qlen - t0);
  const int first_pos = pos0 + t0, last_pos = pos0 + t0 + ntok - 1;
  auto oldest = [&](int p) { return (window > 0 && p - window + 1 > 0) ? p - window + 1 : 0; };
  const int kmin = oldest(first_pos), kend = last_pos + 1;
  const int tile_lo = kmin / SK_BN, tile_hi = (kend + SK_BN - 1) / SK_BN;
  const int keep = window > 0 ? keep_first : 0;
  const int keep_tiles = min((min(keep, kmin) + SK_BN - 1) / SK_BN, tile_lo);
  const int ntiles = keep_tiles + tile_hi - tile_lo;
  auto tile_at = [&](int it) { return it < keep_tiles ? it : tile_lo + it - keep_tiles; };
  const int* bt = block_table + (size_t)s * max_blocks;

  // rows of V that no box fills (pages that are skipped) must hold finite numbers: clear the ring once
  for (int i = threadIdx.x; i < VST * VSTAGE / 16; i += blockDim.x) ((uint4*)sV)[i] = make_uint4(0u, 0u, 0u, 0u);
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < KST; ++i) { mbar_init(&k_full[i], NP); mbar_init(&k_empty[i], 1); }
    for (int i = 0; i < VST; ++i) { mbar_init(&v_full[i], NP); mbar_init(&v_empty[i], 1); }
    mbar_init(s_full, 1);
    mbar_init(p_full, 8);
    mbar_init(pv_full, 1);
    mbar_init(s_free, 8);
    for (int i = 0; i < 4; ++i) mbar_init(&xbar[i], 2);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"((unsigned long long)&map_q) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"((unsigned long long)&map_k) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"((unsigned long long)&map_v) : "memory");
  }
  if (warp == NP) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tg_smem(tmem_slot)), "r"(TMEM) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // the cleared ring, before TMA writes into it
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const unsigned tmem_s = *tmem_slot, tmem_o = tmem_s + SK_BN, tmem_p = tmem_o + DV;   // BN + DV + BN / 2 + 4 <= TMEM columns

  if (warp < NP) {
    // ---- producers: warp w brings pages w, w + NP, ... of every tile, lane l the l-th of them
    if (warp == 0 && lane == 0) {
      mbar_expect_tx(q_full, (unsigned)(panels * bq * g * 128));
      for (int pn = 0; pn < panels; ++pn) tma_load_3d(sQ + pn * 16384, &map_q, pn * 64, kvh * g, qs + t0, q_full);
    }
    const int tile_pages = SK_BN / page_size;
    const int mine = warp + lane * NP;              // this lane's page of a tile
    // the page's number: -1 nothing to bring
    auto fetch = [&](int it) {
      if (mine >= tile_pages || it >= ntiles) return -1;
      const int j = tile_at(it) * SK_BN + mine * page_size;
      if (j >= kend) return -1;
      const int page = bt[j / page_size];
      if (page >= 0 && page < num_pages) return page;
      if (j + page_size > kmin || j < keep) atomicOr(err, 4);      // a page with visible keys is missing
      return -1;
    };
    auto bring = [&](unsigned char* dst, const CUtensorMap* map, int x, int page, unsigned long long* full) {
      const unsigned have = __ballot_sync(0xffffffffu, page >= 0);
      if (lane == 0) mbar_expect_tx(full, (unsigned)(__popc(have) * page_size * 128));
      __syncwarp();
      if (page >= 0) tma_load_2d(dst + mine * page_size * 128, map, x, page * page_size, full);
    };
    bool ok = true;
    int kc = 0, prev = -1, cur = fetch(0);
    // K of a tile, then V of the tile ahead of it: the order in which the products take them
    for (int it = 0; it <= ntiles && ok; ++it) {
      const int next = fetch(it + 1);               // on its way while this tile's boxes are asked for
      if (it < ntiles) {
        for (int pn = 0; pn < panels && ok; ++pn, ++kc) {
          const int st = kc % KST;
          ok = __all_sync(0xffffffffu, mbar_wait(&k_empty[st], ((kc / KST) & 1) ^ 1, err));
          if (ok) bring(sK + st * SK_PANEL, &map_k, pn * 64, cur, &k_full[st]);
        }
      }
      if (it > 0 && ok) {
        const int v = it - 1, st = v % VST;
        ok = __all_sync(0xffffffffu, mbar_wait(&v_empty[st], ((v / VST) & 1) ^ 1, err));
        if (ok) {
          const unsigned have = __ballot_sync(0xffffffffu, prev >= 0);
          if (lane == 0) mbar_expect_tx(&v_full[st], (unsigned)(__popc(have) * page_size * 128 * DP));
          __syncwarp();
          if (prev >= 0)
            for (int pn = 0; pn < DP; ++pn)
              tma_load_2d(sV + st * VSTAGE + pn * SK_PANEL + mine * page_size * 128, &map_v, kvh * DV + pn * 64,
                          prev * page_size, &v_full[st]);
        }
      }
      prev = cur;
      cur = next;
    }
    __syncwarp();
  } else if (warp == NP) {
    if (lane == 0) {
      const unsigned idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((unsigned)(SK_BN >> 3) << 17) | ((unsigned)(SK_BM >> 4) << 24);
      const unsigned idesc_pv = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((unsigned)(DV >> 3) << 17) | ((unsigned)(SK_BM >> 4) << 24);
      const unsigned long long dq = umma_desc(sQ);
      int kc = 0;
      bool ok = mbar_wait(q_full, 0, err);
      // the scores of the next tile, panel by panel as they come in
      auto scores = [&]() {
        for (int pn = 0; pn < panels; ++pn, ++kc) {
          const int st = kc % KST;
          if (!mbar_wait(&k_full[st], (kc / KST) & 1, err)) return false;
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
          const unsigned long long a = dq + (unsigned long long)(pn * (16384 >> 4)), b = umma_desc(sK + st * SK_PANEL);
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16(tmem_s, a + (unsigned long long)(2 * k), b + (unsigned long long)(2 * k), idesc_s, (pn | k) != 0);
          umma_commit(&k_empty[st]);
        }
        umma_commit(s_full);
        return true;
      };
      if (ok) ok = scores();
      for (int it = 0; it < ntiles && ok; ++it) {
        if (it + 1 < ntiles) {
          ok = mbar_wait(s_free, it & 1, err);      // the softmax warps hold this tile's scores
          if (!ok) break;
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
          ok = scores();
          if (!ok) break;
        }
        const int st = it % VST;
        ok = mbar_wait(&v_full[st], (it / VST) & 1, err) && mbar_wait(p_full, it & 1, err);   // P is there, O is rescaled
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        // V is the MN-major operand: 8 keys on 1024 bytes further (stride field), 64 values on a panel further
        const unsigned long long dvd = (umma_desc(sV + st * VSTAGE) & ~(0x3FFFull << 16)) | ((unsigned long long)(SK_PANEL >> 4) << 16);
#pragma unroll
        for (int kk = 0; kk < SK_BN / 16; ++kk)
          umma_bf16_tmem_a(tmem_o, tmem_p + kk * 8, dvd + (unsigned long long)(kk * (2048 >> 4)), idesc_pv, (it | kk) != 0);
        umma_commit(pv_full);
        umma_commit(&v_empty[st]);
      }
    }
    __syncwarp();
  } else {
    // ---- softmax: two threads a row; warp w and w + 4 own the same 32 rows
    const int quarter = warp & 3, half = (warp - NP - 1) >> 2;
    const int r = quarter * 32 + lane;
    const int tl = r / g, hl = r - tl * g;
    const bool live = tl < ntok;
    const int pos = pos0 + t0 + tl;
    const int row_hi = pos + 1, row_lo = oldest(pos);
    const int clear_lo = oldest(pos0 + t0 + bq - 1), clear_hi = first_pos + 1;   // tiles inside need no mask
    float m_ref = -INFINITY, l = 0.f;
    const unsigned lane_sel = (unsigned)(quarter * 32) << 16;
    constexpr int HC = SK_BN / 2;                    // keys a thread
    const unsigned x_mine = tmem_p + SK_BN / 2 + lane_sel + half * 2, x_theirs = tmem_p + SK_BN / 2 + lane_sel + (half ^ 1) * 2;
    bool ok = true;
    for (int it = 0; it < ntiles; ++it) {
      const int j0 = tile_at(it) * SK_BN;
      ok = __all_sync(0xffffffffu, mbar_wait(s_full, it & 1, err));
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      float sc[HC];
#pragma unroll
      for (int c0 = 0; c0 < HC; c0 += 32) tmem_ld32(tmem_s + lane_sel + half * HC + c0, (unsigned*)(sc + c0));
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(s_free);            // the scores are in registers: the next tile's may come
      if (!(j0 >= clear_lo && j0 + SK_BN <= clear_hi)) {
        const unsigned lo_rel = (unsigned)(row_lo - j0 - half * HC), span = (unsigned)(row_hi - row_lo);
        const int keep_rel = min(keep, row_hi) - j0 - half * HC;        // keys below it are kept first keys
#pragma unroll
        for (int j = 0; j < HC; ++j)
          if (!((unsigned)j - lo_rel < span || j < keep_rel)) sc[j] = -INFINITY;
      }
      float mx0 = fmaxf(sc[0], sc[1]), mx1 = fmaxf(sc[2], sc[3]), mx2 = fmaxf(sc[4], sc[5]), mx3 = fmaxf(sc[6], sc[7]);
#pragma unroll
      for (int j = 8; j < HC; j += 8) {
        mx0 = at_max3(mx0, sc[j], sc[j + 1]); mx1 = at_max3(mx1, sc[j + 2], sc[j + 3]);
        mx2 = at_max3(mx2, sc[j + 4], sc[j + 5]); mx3 = at_max3(mx3, sc[j + 6], sc[j + 7]);
      }
      float mx = fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)), mx_other;
      ok = pair_exchange(x_mine + (it & 1), x_theirs + (it & 1), &xbar[quarter], it, mx, &mx_other, err);
      if (!ok) break;
      mx = fmaxf(mx, mx_other) * scale_log2;
      const bool moves = mx > m_ref + 8.0f;          // the reference point moves only when the max has grown by 2^8
      float corr = 1.0f;
      if (moves) {
        corr = at_ex2(m_ref - mx);
        m_ref = mx;
        l *= corr;
      }
      const float m_safe = (m_ref == -INFINITY) ? 0.f : m_ref;
      unsigned pk[HC / 2];
      const unsigned long long scale2 = at_pack2(scale_log2, scale_log2), shift2 = at_pack2(-m_safe, -m_safe);
      unsigned long long sum01 = at_pack2(0.f, 0.f), sum23 = sum01;
#pragma unroll
      for (int j = 0; j < HC; j += 4) {
        float x0, x1, x2, x3;
        at_unpack2(at_fma2(at_pack2(sc[j], sc[j + 1]), scale2, shift2), x0, x1);
        at_unpack2(at_fma2(at_pack2(sc[j + 2], sc[j + 3]), scale2, shift2), x2, x3);
        const float p0 = at_ex2(x0), p1 = at_ex2(x1), p2 = at_ex2(x2), p3 = at_ex2(x3);
        sum01 = at_add2(sum01, at_pack2(p0, p1));
        sum23 = at_add2(sum23, at_pack2(p2, p3));
        __nv_bfloat162 h0 = __floats2bfloat162_rn(p0, p1), h1 = __floats2bfloat162_rn(p2, p3);
        pk[j / 2] = *(unsigned*)&h0;
        pk[j / 2 + 1] = *(unsigned*)&h1;
      }
      {
        float a0, a1, a2, a3;
        at_unpack2(sum01, a0, a1);
        at_unpack2(sum23, a2, a3);
        l += (a0 + a1) + (a2 + a3);
      }
      // the product of the tile before has to be through: it read P, and it wrote the output that is rescaled here
      if (it > 0) {
        ok = __all_sync(0xffffffffu, mbar_wait(pv_full, (it - 1) & 1, err));
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        if (__any_sync(0xffffffffu, moves)) {
#pragma unroll
          for (int c0 = 0; c0 < DV / 2; c0 += 32) {
            unsigned v[32];
            tmem_ld32(tmem_o + lane_sel + half * (DV / 2) + c0, v);
            asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
            for (int j = 0; j < 32; ++j) v[j] = __float_as_uint(__uint_as_float(v[j]) * corr);
            tmem_st32(tmem_o + lane_sel + half * (DV / 2) + c0, v);
          }
          asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        }
      }
      if constexpr (HC == 64) tmem_st32(tmem_p + lane_sel + half * (HC / 2), pk);
      else tmem_st16(tmem_p + lane_sel + half * (HC / 2), pk);
      // rows of V at and behind the last visible key were never written by this sequence: cleared ahead of P V
      if (it == ntiles - 1) {
        const int st = it % VST;
        ok = __all_sync(0xffffffffu, mbar_wait(&v_full[st], (it / VST) & 1, err));
        if (!ok) break;
        if (r < SK_BN && j0 + r >= kend) {
#pragma unroll
          for (int dp = 0; dp < DP; ++dp) {
            uint4* vrow = (uint4*)(sV + st * VSTAGE + dp * SK_PANEL + r * 128 + half * 64);
#pragma unroll
            for (int c = 0; c < 4; ++c) vrow[c] = make_uint4(0u, 0u, 0u, 0u);
          }
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      }
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait(pv_full, (ntiles - 1) & 1, err));
    float lother = 0.f;
    if (ok) ok = pair_exchange(x_mine + (ntiles & 1), x_theirs + (ntiles & 1), &xbar[quarter], ntiles, l, &lother, err);
    if (ok) {
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const float lsum = half == 0 ? l + lother : lother + l;
      const float inv = lsum > 0.f ? 1.0f / lsum : 0.f;
      const int head = kvh * g + hl;
      bf16* orow = out + ((size_t)(qs + t0 + tl) * nq + head) * dv;
      const bool vec = (dv & 7) == 0;
#pragma unroll
      for (int c0 = 0; c0 < DV / 2; c0 += 32) {
        const int col = half * (DV / 2) + c0;
        unsigned v[32];
        tmem_ld32(tmem_o + lane_sel + col, v);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        if (live) {
#pragma unroll
          for (int c = 0; c < 32; c += 8) {
            if (vec && col + c + 8 <= dv) {
              uint4 w;
              __nv_bfloat162* h = (__nv_bfloat162*)&w;
#pragma unroll
              for (int q = 0; q < 4; ++q)
                h[q] = __floats2bfloat162_rn(__uint_as_float(v[c + 2 * q]) * inv, __uint_as_float(v[c + 2 * q + 1]) * inv);
              *(uint4*)(orow + col + c) = w;
            } else {
#pragma unroll
              for (int q = 0; q < 8; ++q)
                if (col + c + q < dv) orow[col + c + q] = __float2bfloat16_rn(__uint_as_float(v[c + q]) * inv);
            }
          }
        }
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == NP) {
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_s), "r"(TMEM) : "memory");
  }
}

template <int DV, bool BIG>
static int sk_launch(const void* q, int num_q_rows, void* out, const void* kcache, const void* vcache, const int* block_table,
                     int max_blocks, const int* q_start, const int* seq_lens, int seq_begin, int seq_end, int num_tokens,
                     int nq, int nkv, int dkp, int dv, int page_size, int num_pages, int window, int keep_first, float scale,
                     int* err, cudaStream_t stream) {
  const int g = nq / nkv, panels = dkp / 64;
  CUtensorMap mq, mk, mv;
  {
    cuuint64_t dims[3] = {(cuuint64_t)dkp, (cuuint64_t)nq, (cuuint64_t)num_q_rows};
    cuuint64_t strides[2] = {(cuuint64_t)dkp * 2, (cuuint64_t)nq * dkp * 2};
    cuuint32_t box[3] = {64, (cuuint32_t)g, (cuuint32_t)(SK_BM / g)};
    int rc = at_encode(&mq, 3, q, dims, strides, box);
    if (rc) return rc;
  }
  {
    cuuint64_t dims[2] = {(cuuint64_t)dkp, (cuuint64_t)num_pages * page_size};
    cuuint64_t strides[1] = {(cuuint64_t)dkp * 2};
    cuuint32_t box[2] = {64, (cuuint32_t)page_size};
    int rc = at_encode(&mk, 2, kcache, dims, strides, box);
    if (rc) return rc;
    dims[0] = (cuuint64_t)nkv * DV;
    strides[0] = (cuuint64_t)nkv * DV * 2;
    rc = at_encode(&mv, 2, vcache, dims, strides, box);
    if (rc) return rc;
  }
  const int smem = sk_smem<DV, BIG>(panels);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(shared_key_tcgen05_kernel<DV, BIG>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         sk_smem<DV, BIG>(BIG ? 8 : 4));
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int bq = SK_BM / g;
  const long long tiles = (num_tokens + bq - 1) / bq + (seq_end - seq_begin);
  if (tiles * nkv > 0x7fffffffLL) return RLLM_E_UNSUPPORTED;
  shared_key_tcgen05_kernel<DV, BIG><<<dim3((unsigned)(tiles * nkv)), sk_threads<BIG>(), smem, stream>>>(
      mq, mk, mv, (bf16*)out, block_table, max_blocks, q_start, seq_lens, seq_begin, seq_end, nq, nkv, panels, dv, page_size,
      num_pages, window, keep_first, scale * 1.4426950408889634f, err);
  RLLM_LAUNCH_CHECK();
  return 0;
}

// Sequences seq_begin .. seq_end-1 of the step.  q: num_q_rows rows of nq * dkp (dkp a multiple of 64 up to 512), the rows
// of the sequences' tokens at q_start; keys [pages, 1, page_size, dkp], values [pages, 1, page_size, nkv * dvp] with dvp
// 64 or 128; out [., nq * dv]; pages of 16, 32 or 64 keys; up to 128 query heads a kv head.
RLLM_EXPORT int rllm_shared_key_attention_tcgen05(const void* q, int num_q_rows, void* out, const void* kcache,
                                                  const void* vcache, const int* block_table, int max_blocks,
                                                  const int* q_start, const int* seq_lens, int seq_begin, int seq_end,
                                                  int num_tokens, int nq, int nkv, int dkp, int dv, int dvp, int page_size,
                                                  int num_pages, int window, int keep_first, float scale, int* err,
                                                  cudaStream_t stream) {
  if (seq_end <= seq_begin || num_tokens <= 0) return 0;
  if (nq <= 0 || nkv <= 0 || nq % nkv || num_pages <= 0 || max_blocks <= 0 || window < 0 || keep_first < 0 || dv <= 0 ||
      dv > dvp || !(scale > 0.f) || !err || num_q_rows <= 0)
    return RLLM_E_BADARG;
  if (dkp % 64 || dkp <= 0 || dkp > 512 || !(dvp == 64 || dvp == 128) || !(page_size == 16 || page_size == 32 || page_size == 64) ||
      nq / nkv > SK_BM || (long long)num_pages * page_size > 0x7fffffffLL ||
      (((uintptr_t)q | (uintptr_t)kcache | (uintptr_t)vcache) & 15))
    return RLLM_E_UNSUPPORTED;
#define SK_GO(DV_, BIG_)                                                                                                  \
  return sk_launch<DV_, BIG_>(q, num_q_rows, out, kcache, vcache, block_table, max_blocks, q_start, seq_lens, seq_begin,   \
                              seq_end, num_tokens, nq, nkv, dkp, dv, page_size, num_pages, window, keep_first, scale, err, \
                              stream)
  if (dvp == 64) { if (dkp > 256) SK_GO(64, true); SK_GO(64, false); }
  if (dkp > 256) SK_GO(128, true);
  SK_GO(128, false);
#undef SK_GO
}

// The mma.sync form.  Which warps a CTA takes: eight where keys and values of 64 tokens fit twice in shared memory, else four.
static int sk_mma_warps(int rows, int dkp, int dvt) {
  const int mt = rows <= 16 ? 1 : 2;
  for (int nw = 8; nw >= 4; nw -= 4) {
    const int keys = 8 * nw, cols = dvt <= 64 && nw == 8 ? 64 : (dvt <= 128 && nw == 8 ? 128 : (dvt <= 256 ? 256 : 512));
    const size_t smem = 2 * ((size_t)16 * mt * (dkp + 8) + 2 * keys * (dkp + 8 + cols + 8) + 16 * mt * (keys + 8)) +
                        4 * (size_t)(2 * nw * 16 * mt * 2 + 2 * 16 * mt);
    if (smem <= 220 * 1024) return nw;
  }
  return 0;
}
RLLM_EXPORT int rllm_shared_key_attention_mma_takes(int heads, int dkp, int dvt) {
  return dkp > 0 && dkp % 32 == 0 && dvt > 0 && dvt % 8 == 0 && dvt <= 512 && sk_mma_warps(32, dkp, dvt) > 0 ? 1 : 0;
}
// work in floats for a call with splits
RLLM_EXPORT long long rllm_shared_key_attention_mma_work(int S, int max_q, int heads, int dvp, int nsplit) {
  const long long rows = (long long)max_q * heads;
  const int tile = rows <= 16 ? 16 : 32;
  return (long long)S * ((rows + tile - 1) / tile * tile) * nsplit * (dvp + 2);
}

// Sequences 0 .. S-1, sequence s with the tokens q_start[s] .. q_start[s+1]; max_q: the most tokens one brings.  split_keys
// > 0 (a multiple of 64): the keys in nsplit splits side by side, at least as many as the splits that hold a sequence's
// kept and recent keys.
RLLM_EXPORT int rllm_shared_key_attention_mma(const void* q, void* out, const void* kcache, const void* vcache,
                                              const int* block_table, int max_blocks, const int* q_start,
                                              const int* seq_lens, int S, int max_q, int nq, int nkv, int dkp, int dv,
                                              int dvp, int page_size, int num_pages, int window, int keep_first,
                                              float scale, int split_keys, int nsplit, float* work, int* err,
                                              cudaStream_t stream) {
  if (S <= 0 || max_q <= 0) return 0;
  if (split_keys > 0 && (split_keys % 64 != 0 || nsplit <= 0 || nsplit > 8192 || work == nullptr)) return RLLM_E_BADARG;
  if (nq <= 0 || nkv <= 0 || nq % nkv || dkp <= 0 || dv <= 0 || dv > dvp || page_size <= 0 || num_pages <= 0 ||
      max_blocks <= 0 || window < 0 || keep_first < 0)
    return RLLM_E_BADARG;
  const int dvt = nkv * dvp;
  if (!rllm_shared_key_attention_mma_takes(nq, dkp, dvt) || dvp % 2 ||
      (((uintptr_t)q | (uintptr_t)kcache | (uintptr_t)vcache) & 15) != 0 || ((uintptr_t)out & 3) != 0)
    return RLLM_E_UNSUPPORTED;
  const long long rows = (long long)max_q * nq;
  const int nw = sk_mma_warps(rows <= 16 ? 16 : 32, dkp, dvt);
#define SKM_GO(MT_, NVT_, NW_)                                                                                            \
  return lam_launch<MT_, NVT_, NW_, true>((const bf16*)q, (bf16*)out, (const bf16*)kcache, block_table, max_blocks, q_start, \
                                          seq_lens, S, max_q, nq, dkp, dv, page_size, num_pages, window, scale, nullptr,   \
                                          split_keys, nsplit, work, err, stream,                                          \
                                          LamSep{(const bf16*)vcache, nkv, dvp, keep_first})
#define SKM_PICK(NVT_, NW_)                              \
  do {                                                   \
    if (rows <= 16) SKM_GO(1, NVT_, NW_);                \
    SKM_GO(2, NVT_, NW_);                                \
  } while (0)
  if (nw == 8) {
    if (dvt <= 64) SKM_PICK(1, 8);
    if (dvt <= 128) SKM_PICK(2, 8);
    if (dvt <= 256) SKM_PICK(4, 8);
    SKM_PICK(8, 8);
  }
  if (dvt <= 256) SKM_PICK(8, 4);
  SKM_PICK(16, 4);
#undef SKM_PICK
#undef SKM_GO
}
