// Paged causal attention over latents on the 5th-generation tensor cores (bfloat16): one shared key
// row per token, of up to about 700 channels, whose first `vdim` channels are the value.
//
// With one key head every (token, query head) pair of a request is one more row of the same
// problem, so the queries are taken as a matrix of flat rows [tokens * heads][key channels] and a
// CTA takes up to 128 consecutive ones, whatever the number of heads, one TMEM lane each.  A row's
// position is that of its token.  The product takes 128 rows whatever a CTA has; where it has
// fewer (steps of single tokens), only
// theirs are kept in shared memory and the product's other rows read what lies behind them: their
// results are not used.  Keys are walked in tiles of 64 aligned to absolute positions.
// Channels are cut into blocks of 64 (128 bytes, one swizzle span; the last block is filled with
// zeros).  A tile's blocks that are also values of this CTA ("value blocks", at most four: 256
// accumulator columns) stay in shared memory until the second product has read them; the other
// blocks pass, in groups, through a ring of their own and are free once the scores have read them.  With more
// value blocks than a CTA takes, several CTAs share the same rows, each with its part of the value
// channels; they make the scores anew.  The keys can be cut into `splits` parts whose results a merge
// kernel joins (steps of few rows).
//
//   warp 0     TMA: the query rows once (a box per block of channels), then the blocks of keys that
//              are no values of this CTA, tile by tile
//   warp 6     TMA: the value blocks, tile by tile
//   warp 1     one lane issues  S = Q K^T  into one of two TMEM score buffers and  O += P V  (A = P from
//              TMEM, B = the value blocks, N-major), in the order S0, S1, PV0, S2, PV1, ...
//   warps 2-5  softmax, one thread per row: scores into registers, maximum, exponentials and sum in
//              32-bit, P back as bfloat16 over the scores; the output is rescaled only when a row's
//              maximum has grown by more than 2^8 since the scale in use; finally O / l is written,
//              with the sink as one more entry of the sum, or (splits) O, the maximum and l as a part
//
// Every mbarrier wait is bounded; when one gives up the kernel records where in *status, lets its
// loads land, frees its TMEM and returns.
#include "attention_tc_common.cuh"

namespace {

constexpr int ROWS = 128;             // flat rows of a CTA (TMEM lanes)
constexpr int MAX_VS = 4, MAX_XS = 8;  // most stages of value blocks, of groups of other blocks
constexpr int KT = 64;                // keys per tile
constexpr int KBLK = KT * 128;        // bytes of a block of 64 channels of a tile's keys
constexpr int SMEM_LIMIT = 227 * 1024;

struct Bars {
  uint64_t q_full;
  uint64_t v_full[MAX_VS], v_empty[MAX_VS];
  uint64_t x_full[MAX_XS], x_empty[MAX_XS];
  uint64_t s_full[2], p_full[2];
  uint64_t o_done;
  uint32_t tmem_base;
  int dead;
  int stop[2];
};

struct LatentArgs {
  const int* block_table; int table_stride;
  const int* items;           // device (first flat row, flat rows, request slot, 0), or null: see `per_row`
  int per_row;                // without items: CTAs of flat rows per token (every request has one token)
  const int* row_pos;
  const int* row_slot;
  long long rows_per_page;
  int q_rows;                 // rows of queries in shared memory (a multiple of 8)
  int H, page_size, kd_blocks, vdim, v_blocks, chunks, vs, xs, xg, tmem_cols;
  float scale_log2;
  int window, splits;
  bf16* out;                  // [flat rows][vdim]
  float* part_o;              // [flat rows][splits][vdim]
  float* part_ml;             // [flat rows][splits][chunks][2]
  const float* sink;
  int* status;
};

__global__ void __launch_bounds__(224, 1) attention_latent_kernel(const __grid_constant__ CUtensorMap map_q,
                                                                  const __grid_constant__ CUtensorMap map_k,
                                                                  const LatentArgs a) {
  constexpr uint32_t O_COL = 2 * KT;
  constexpr uint32_t IDESC_S = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(KT >> 3) << 17) |
                               ((uint32_t)(ROWS >> 4) << 24);
  extern __shared__ uint8_t raw[];
  uint8_t* base_s = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~(uintptr_t)1023);
  const int nkb = a.kd_blocks;
  const uint32_t QBLK = (uint32_t)a.q_rows * 128;            // bytes of a block of 64 channels of the queries
  uint8_t* q_s = base_s;                                     // [nkb][q_rows][128 bytes]
  uint8_t* v_s = q_s + (size_t)nkb * QBLK;                   // [vs][v_blocks][64 keys][128 bytes]
  uint8_t* x_s = v_s + (size_t)a.vs * a.v_blocks * KBLK;     // [xs][xg][64 keys][128 bytes]
  Bars& sm = *reinterpret_cast<Bars*>(x_s + (size_t)a.xs * a.xg * KBLK);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // the last items of a prompt have the most keys to walk: they are started first
  const int n_items = gridDim.x / a.chunks;
  const int item = n_items - 1 - blockIdx.x / a.chunks, chunk = blockIdx.x % a.chunks;
  const int split = blockIdx.y;
  const int vb0 = chunk * a.v_blocks;                        // first value block of this CTA
  const int vcap = (a.vdim + 63) / 64;                       // blocks that hold values
  const int nv = min(a.v_blocks, vcap - vb0);
  const int nx = nkb - nv;

  if (threadIdx.x == 0) {
    mbar_init(&sm.q_full, 1);
    for (int s = 0; s < a.vs; ++s) mbar_init(&sm.v_full[s], 1), mbar_init(&sm.v_empty[s], 1);
    for (int s = 0; s < a.xs; ++s) mbar_init(&sm.x_full[s], 1), mbar_init(&sm.x_empty[s], 1);
    for (int b = 0; b < 2; ++b) mbar_init(&sm.s_full[b], 1), mbar_init(&sm.p_full[b], 4);
    mbar_init(&sm.o_done, 1);
    sm.dead = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm.tmem_base)),
                 "r"((uint32_t)a.tmem_cols)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (warp >= 2) {
    // a page without a key of the item is not fetched and leaves what the stage held; as values
    // these meet zero weights and must be finite: start from zeros
    uint4* v4 = reinterpret_cast<uint4*>(v_s);
    for (int i = threadIdx.x - 64; i < a.vs * a.v_blocks * (KBLK / 16); i += 160) v4[i] = make_uint4(0, 0, 0, 0);
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm.tmem_base;
  pdl_trigger();             // after the allocation: a successor that also allocates cannot starve this CTA
  pdl_wait();

  // the item (positions and slots of the step are written by the host's copy in front of it)
  int f0, nf, slot;
  if (a.items) {
    const Item it = reinterpret_cast<const Item*>(a.items)[item];
    f0 = it.row_start, nf = it.tokens, slot = it.slot;
  } else {
    const int row = item / a.per_row, part = item % a.per_row;
    f0 = row * a.H + part * ROWS, nf = min(ROWS, a.H - part * ROWS), slot = a.row_slot[row];
  }
  const int pos_first = a.row_pos[f0 / a.H], pos_last = a.row_pos[(f0 + nf - 1) / a.H];
  const int lo = first_key(pos_first, a.window), hi = pos_last;
  int tile_first = lo / KT, ntiles = hi / KT - tile_first + 1;
  {
    const int per = (ntiles + a.splits - 1) / a.splits;
    const int t0 = min(ntiles, split * per), t1 = min(ntiles, t0 + per);
    tile_first += t0, ntiles = t1 - t0;
  }
  const int R = min(a.page_size, KT);
  const int* table = a.block_table + (size_t)slot * a.table_stride;
  // Where a tile's keys lie: the row of the key matrix for each page it touches, -1 for a page without
  // a key of the item (it may be gone).  Looked up a tile ahead of the loads that use it.
  struct TileRows { int row[KT / 8]; int live; };
  const int pieces = KT / R;
  auto look_up = [&](int base, TileRows& t) {
    t.live = 0;
#pragma unroll
    for (int g = 0; g < KT / 8; ++g) {
      t.row[g] = -1;
      const int p = base + g * R;
      if (g < pieces && p <= hi && p + R - 1 >= lo) {
        const int page = p / a.page_size;
        t.row[g] = (int)((long long)table[page] * a.rows_per_page + (p - page * a.page_size));
        t.live += R;
      }
    }
  };
  // one block of 64 channels of a tile's keys: a box per page
  auto load_block = [&](uint8_t* dst, int kb, const TileRows& t, uint64_t* bar) {
    if (pieces == 1) {
      tma_load_2d(dst, &map_k, kb * 64, t.row[0], bar);
      return;
    }
#pragma unroll
    for (int g = 0; g < KT / 8; ++g)
      if (t.row[g] >= 0) tma_load_2d(dst + g * R * 128, &map_k, kb * 64, t.row[g], bar);
  };

  if (ntiles > 0) {
    if (warp == 0 && lane == 0) {
      // ---------------------------------------------------------------- queries, blocks that are no values
      mbar_expect_tx(&sm.q_full, (uint32_t)nkb * QBLK);
      for (int kb = 0; kb < nkb; ++kb) tma_load_2d(q_s + (size_t)kb * QBLK, &map_q, kb * 64, f0, &sm.q_full);
      bool ok = true;
      int s = 0, n = 0;                 // the next stage of the ring; groups issued
      uint32_t phase = 0;               // flips whenever the ring has gone round
      TileRows now, next;
      if (nx > 0) look_up(tile_first * KT, next);
      for (int j = 0; j < ntiles && nx > 0 && ok; ++j) {
        now = next;
        const uint32_t bytes = (uint32_t)now.live * 128;
        for (int x0 = 0; x0 < nx; x0 += a.xg) {
          ok = mbar_wait(&sm.x_empty[s], phase ^ 1);
          if (!ok) { atomicExch(a.status, 5); *(volatile int*)&sm.dead = 1; break; }
          const int g = min(a.xg, nx - x0);
          mbar_expect_tx(&sm.x_full[s], bytes * g);
          for (int x = x0; x < x0 + g; ++x)
            load_block(x_s + (size_t)(s * a.xg + x - x0) * KBLK, x < vb0 ? x : x + nv, now, &sm.x_full[s]);
          ++n;
          if (++s == a.xs) s = 0, phase ^= 1;
        }
        if (j + 1 < ntiles) look_up((tile_first + j + 1) * KT, next);
      }
      if (!ok) {     // let what is in flight land before the shared memory is given up
        mbar_wait(&sm.q_full, 0);
        for (int i = max(0, n - a.xs); i < n; ++i)
          mbar_wait(&sm.x_full[i % a.xs], (uint32_t)((i / a.xs) & 1));
      }
    } else if (warp == 6 && lane == 0) {
      // ---------------------------------------------------------------- value blocks
      bool ok = true;
      int j = 0, s = 0;
      uint32_t phase = 0;
      TileRows now, next;
      look_up(tile_first * KT, next);
      for (; j < ntiles; ++j) {
        now = next;
        ok = mbar_wait(&sm.v_empty[s], phase ^ 1);
        if (!ok) { atomicExch(a.status, 5); *(volatile int*)&sm.dead = 1; break; }
        mbar_expect_tx(&sm.v_full[s], (uint32_t)(now.live * 128 * nv));
        for (int b = 0; b < nv; ++b)
          load_block(v_s + (size_t)(s * a.v_blocks + b) * KBLK, vb0 + b, now, &sm.v_full[s]);
        if (++s == a.vs) s = 0, phase ^= 1;
        if (j + 1 < ntiles) look_up((tile_first + j + 1) * KT, next);
      }
      if (!ok)
        for (int i = max(0, j - a.vs); i < j; ++i) mbar_wait(&sm.v_full[i % a.vs], (uint32_t)((i / a.vs) & 1));
    } else if (warp == 1 && lane == 0) {
      // ---------------------------------------------------------------- MMA issuer
      const uint32_t idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(nv * 64 >> 3) << 17) |
                               ((uint32_t)(ROWS >> 4) << 24);
      bool ok = mbar_wait(&sm.q_full, 0);
      if (!ok) { atomicExch(a.status, 6); *(volatile int*)&sm.dead = 1; }
      int xstage = 0, vstage = 0, pstage = 0;          // stages of the rings: other blocks, values for S, for PV
      uint32_t xphase = 0, vphase = 0;
      const uint64_t q_desc = smem_desc(smem_u32(q_s));
      const uint32_t x_addr = smem_u32(x_s), v_addr = smem_u32(v_s), v_stage = (uint32_t)a.v_blocks * KBLK;
      auto scores = [&](uint32_t acc, int kb, uint32_t blk, bool first) {
        const uint64_t qd = q_desc + (uint64_t)((uint32_t)kb * QBLK >> 4), kd = smem_desc(blk);
#pragma unroll
        for (int ks = 0; ks < 4; ++ks)
          tc_mma(acc, qd + (uint64_t)(ks * 2), kd + (uint64_t)(ks * 2), IDESC_S, (first && ks == 0) ? 0u : 1u);
      };
      for (int j = 0; j <= ntiles && ok; ++j) {
        if (j < ntiles) {
          const uint32_t acc = tmem + (uint32_t)(j & 1) * KT;
          for (int x0 = 0; x0 < nx; x0 += a.xg) {
            ok = mbar_wait(&sm.x_full[xstage], xphase);
            if (!ok) break;
            tc_fence_after();
            for (int x = x0; x < min(nx, x0 + a.xg); ++x)
              scores(acc, x < vb0 ? x : x + nv, x_addr + (uint32_t)(xstage * a.xg + x - x0) * KBLK, x == 0);
            tc_commit(&sm.x_empty[xstage]);
            if (++xstage == a.xs) xstage = 0, xphase ^= 1;
          }
          ok = ok && mbar_wait(&sm.v_full[vstage], vphase);
          if (!ok) { atomicExch(a.status, 6); *(volatile int*)&sm.dead = 1; break; }
          tc_fence_after();
          for (int b = 0; b < nv; ++b)
            scores(acc, vb0 + b, v_addr + (uint32_t)vstage * v_stage + (uint32_t)b * KBLK, nx == 0 && b == 0);
          if (++vstage == a.vs) vstage = 0, vphase ^= 1;
          tc_commit(&sm.s_full[j & 1]);
        }
        if (j >= 1) {
          const int i = j - 1;
          ok = mbar_wait(&sm.p_full[i & 1], (uint32_t)((i >> 1) & 1));
          if (!ok) { atomicExch(a.status, 6); *(volatile int*)&sm.dead = 1; break; }
          tc_fence_after();
          const uint32_t p_addr = tmem + (uint32_t)(i & 1) * KT;       // P over the first KT / 2 columns
          const uint32_t va = v_addr + (uint32_t)pstage * v_stage;
#pragma unroll
          for (int ks = 0; ks < KT / UMMA_K; ++ks)
            tc_mma_ts(tmem + O_COL, p_addr + (uint32_t)ks * (UMMA_K / 2), smem_desc_mn(va + (uint32_t)ks * UMMA_K * 128, KBLK),
                      idesc_o, (i > 0 || ks > 0) ? 1u : 0u);
          tc_commit(&sm.v_empty[pstage]);
          tc_commit(&sm.o_done);
          if (++pstage == a.vs) pstage = 0;
        }
      }
    } else if (warp >= 2 && warp < 6) {
      // ---------------------------------------------------------------- softmax
      const int q4 = warp & 3;
      const int row = q4 * 32 + lane;
      const uint32_t lane_base = (uint32_t)(q4 * 32) << 16;
      const bool rvalid = row < nf;
      const int flat = f0 + (rvalid ? row : 0);
      const int tok = flat / a.H, head = flat - tok * a.H;
      const int rpos = a.row_pos[tok];
      const int rlo = first_key(rpos, a.window);
      const bool warp_idle = q4 * 32 >= nf;
      float m_used = -INFINITY, l = 0.f;
      bool ok = true;
      for (int j = 0; j < ntiles; ++j) {
        const int b = j & 1;
        ok = mbar_wait(&sm.s_full[b], (uint32_t)((j >> 1) & 1));
        if (!ok) { if (lane == 0) atomicExch(a.status, 7); *(volatile int*)&sm.dead = 1; }
        // All softmax warps go on or all stop: one thread copies the flag before the barrier and
        // all read the copy behind it.
        if (threadIdx.x == 64) *(volatile int*)&sm.stop[b] = *(volatile int*)&sm.dead;
        asm volatile("bar.sync 1, 128;" ::: "memory");
        if (*(volatile int*)&sm.stop[b]) { ok = false; break; }
        tc_fence_after();
        if (warp_idle) {       // no row of the item: what the products make of these lanes is not used
          if (lane == 0) mbar_arrive(&sm.p_full[b]);
          continue;
        }
        const uint32_t s_addr = tmem + lane_base + (uint32_t)b * KT;
        const int base = (tile_first + j) * KT;
        // (a lane without a row of the item takes the first row's place; its result is not written)
        const int c_hi = min(KT - 1, rpos - base);
        const int c_lo = max(0, rlo - base);
        // a tile that every row of the CTA sees completely needs no per-key tests
        const bool interior = base + KT - 1 <= pos_first && base >= first_key(hi, a.window);
        uint32_t v[KT];
#pragma unroll
        for (int c = 0; c < KT; c += 32) tmem_ld32(s_addr + c, v + c);
        tmem_ld_wait();
        if (!interior) {
#pragma unroll
          for (int c = 0; c < KT; c += 32) {
            // a bit per column: those from c_lo on, up to c_hi
            const int n_hi = c_hi + 1 - c, n_lo = c_lo - c;
            const uint32_t up_to = n_hi <= 0 ? 0u : n_hi >= 32 ? ~0u : (1u << n_hi) - 1u;
            const uint32_t below = n_lo <= 0 ? 0u : n_lo >= 32 ? ~0u : (1u << n_lo) - 1u;
            const uint32_t seen = up_to & ~below;
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (!(seen & (1u << i))) v[c + i] = 0xff800000u;      // -inf: the key is not visible
          }
        }
        float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int i = 0; i < KT; i += 4) {
          mx[0] = fmaxf(mx[0], __uint_as_float(v[i]));
          mx[1] = fmaxf(mx[1], __uint_as_float(v[i + 1]));
          mx[2] = fmaxf(mx[2], __uint_as_float(v[i + 2]));
          mx[3] = fmaxf(mx[3], __uint_as_float(v[i + 3]));
        }
        const float m_tile = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * a.scale_log2;
        const bool grow = m_tile > m_used + 8.0f;
        float factor = 1.f;
        if (grow) {
          factor = m_used == -INFINITY ? 0.f : ex2(m_used - m_tile);
          m_used = m_tile;
          l *= factor;
        }
        if (j > 0 && __any_sync(0xffffffffu, grow)) {
          // rare once the maximum has settled: the rows of this warp in O are rescaled, for which
          // the product P V of the tile before must be complete
          const bool done = mbar_wait(&sm.o_done, (uint32_t)((j - 1) & 1));
          if (!done) { if (lane == 0) atomicExch(a.status, 7); *(volatile int*)&sm.dead = 1; }
          tc_fence_after();
#pragma unroll 1
          for (int c = 0; c < nv * 64; c += 32) {
            uint32_t w[32];
            tmem_ld32(tmem + lane_base + O_COL + c, w);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) w[i] = __float_as_uint(__uint_as_float(w[i]) * factor);
            tmem_st32(tmem + lane_base + O_COL + c, w);
          }
          tmem_st_wait();
        }
        const float muse = m_used == -INFINITY ? 0.f : m_used;
#pragma unroll
        for (int i = 0; i < KT; ++i)
          v[i] = __float_as_uint(ex2(fmaf(__uint_as_float(v[i]), a.scale_log2, -muse)));
        float sum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < KT; i += 4) {
          sum[0] += __uint_as_float(v[i]);
          sum[1] += __uint_as_float(v[i + 1]);
          sum[2] += __uint_as_float(v[i + 2]);
          sum[3] += __uint_as_float(v[i + 3]);
        }
        l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
#pragma unroll
        for (int c = 0; c < KT; c += 32) {
          uint32_t pk[16];
#pragma unroll
          for (int i = 0; i < 32; i += 2)
            pk[i >> 1] = pack2(__uint_as_float(v[c + i]), __uint_as_float(v[c + i + 1]));
          tmem_st16(s_addr + (c >> 1), pk);
        }
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&sm.p_full[b]);
      }
      if (ok && !warp_idle) {
        bool done = mbar_wait(&sm.o_done, (uint32_t)((ntiles - 1) & 1));
        if (!done) { if (lane == 0) atomicExch(a.status, 7); }
        done = __all_sync(0xffffffffu, done);
        if (done) {
          tc_fence_after();
          const bool parts = a.splits > 1;
          float inv = 1.f;
          if (!parts) {
            // the sink: one more entry of the sum that has no value (m_used is a base-2 logarithm,
            // finite for a row that sees its own key)
            if (a.sink && rvalid) {
              const float z = a.sink[head] * 1.4426950408889634f;
              const float m = fmaxf(z, m_used);
              l = l * ex2(m_used - m) + ex2(z - m);
              inv = ex2(m_used - m) / l;
            } else {
              inv = 1.f / l;
            }
          } else if (rvalid) {
            // (every CTA of a group of rows has a maximum and a sum of its own: it makes the scores
            // from the same blocks in another order)
            float* ml = a.part_ml + (((size_t)flat * a.splits + split) * a.chunks + chunk) * 2;
            ml[0] = m_used, ml[1] = l;
          }
          const int c_begin = vb0 * 64;
          bf16* dst = a.out + (size_t)flat * a.vdim + c_begin;
          float* pdst = a.part_o + ((size_t)flat * a.splits + split) * a.vdim + c_begin;
          const int width = min(nv * 64, a.vdim - c_begin);
          const bool wide = (a.vdim & 7) == 0;
#pragma unroll 1
          for (int c = 0; c < nv * 64; c += 32) {
            uint32_t w[32];
            tmem_ld32(tmem + lane_base + O_COL + c, w);
            tmem_ld_wait();
            if (!rvalid) {
            } else if (parts) {
              if (wide) {
#pragma unroll
                for (int i = 0; i < 32; i += 4)
                  if (c + i < width)
                    *reinterpret_cast<uint4*>(pdst + c + i) = make_uint4(w[i], w[i + 1], w[i + 2], w[i + 3]);
              } else {
#pragma unroll
                for (int i = 0; i < 32; ++i)
                  if (c + i < width) pdst[c + i] = __uint_as_float(w[i]);
              }
            } else if (wide) {
#pragma unroll
              for (int i = 0; i < 32; i += 8) {
                if (c + i >= width) continue;
                uint4 u;
                u.x = pack2(__uint_as_float(w[i]) * inv, __uint_as_float(w[i + 1]) * inv);
                u.y = pack2(__uint_as_float(w[i + 2]) * inv, __uint_as_float(w[i + 3]) * inv);
                u.z = pack2(__uint_as_float(w[i + 4]) * inv, __uint_as_float(w[i + 5]) * inv);
                u.w = pack2(__uint_as_float(w[i + 6]) * inv, __uint_as_float(w[i + 7]) * inv);
                *reinterpret_cast<uint4*>(dst + c + i) = u;
              }
            } else {
#pragma unroll
              for (int i = 0; i < 32; ++i)
                if (c + i < width) dst[c + i] = __float2bfloat16_rn(__uint_as_float(w[i]) * inv);
            }
            __syncwarp();
          }
        }
      }
    }
  } else if (warp >= 2 && warp < 6) {
    // a part without keys: the merge passes over it
    const int row = (warp & 3) * 32 + lane;
    if (row < nf) {
      float* ml = a.part_ml + (((size_t)(f0 + row) * a.splits + split) * a.chunks + chunk) * 2;
      ml[0] = -INFINITY, ml[1] = 0.f;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"((uint32_t)a.tmem_cols)
                 : "memory");
  }
}

// out[f][:] = sum over the parts of a flat row, with the sink as a part without an output; block
// (f, c) makes the channels of the c-th CTA of the row's group.  A part whose maximum is -inf has no
// keys; its output was not written.
__global__ void __launch_bounds__(128) attention_latent_merge_kernel(const float* __restrict__ part_o,
                                                                     const float* __restrict__ part_ml,
                                                                     bf16* __restrict__ out, int H, int vdim,
                                                                     int splits, int per_chunk,
                                                                     const float* __restrict__ sink) {
  extern __shared__ float w_s[];        // a weight per part
  pdl_trigger();
  pdl_wait();
  const size_t f = blockIdx.x;
  const int chunk = blockIdx.y, step = 2 * gridDim.y;
  const float* ml = part_ml + (f * splits * gridDim.y + chunk) * 2;
  if (threadIdx.x < 32) {
    const float z = sink ? sink[f % H] * 1.4426950408889634f : -INFINITY;
    float m = z;
    for (int s = threadIdx.x; s < splits; s += 32) m = fmaxf(m, ml[step * s]);
    m = warp_max(m);
    float l = 0.f;
    for (int s = threadIdx.x; s < splits; s += 32) {
      const float w = ml[step * s] == -INFINITY ? 0.f : ex2(ml[step * s] - m);
      w_s[s] = w;
      l += w * ml[step * s + 1];
    }
    l = warp_sum(l);
    if (sink) l += ex2(z - m);
    __syncwarp();
    for (int s = threadIdx.x; s < splits; s += 32) w_s[s] /= l;
  }
  __syncthreads();
  const float* o = part_o + f * splits * vdim;
  for (int c = chunk * per_chunk + threadIdx.x; c < min(vdim, (chunk + 1) * per_chunk); c += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < splits; ++s)
      if (w_s[s] != 0.f) acc = fmaf(w_s[s], o[(size_t)s * vdim + c], acc);
    out[f * vdim + c] = __float2bfloat16_rn(acc);
  }
}

// how the shared memory of a CTA is laid out for these sizes; false: they do not fit
struct Layout { int kd_blocks, chunks, v_blocks, vs, xs, xg, smem, tmem_cols, q_rows; };
bool layout_for(int kd, int vdim, int q_rows, Layout* L) {
  const int QBLK = q_rows * 128;
  const int nkb = (kd + 63) / 64, ncb = (vdim + 63) / 64;
  const int room = SMEM_LIMIT - 1024 - (int)sizeof(Bars) - nkb * QBLK;
  for (int chunks = (ncb + 3) / 4; chunks <= ncb; ++chunks) {
    const int nv = (ncb + chunks - 1) / chunks;
    if ((ncb + nv - 1) / nv != chunks) continue;       // (an empty last chunk)
    // blocks of a CTA that are no values (the last CTA may have fewer value blocks than the others)
    const int others = nkb - (ncb - (chunks - 1) * nv);
    int vs = 2, xs = others ? 2 : 1, xg = 1;
    if ((vs * nv + xs) * KBLK > room) continue;
    // as few groups as two stages of them fit: every group costs the issuing thread a wait
    while (xg < others && (vs * nv + xs * (xg + 1)) * KBLK <= room) ++xg;
    if (others) xg = (others + (others + xg - 1) / xg - 1) / ((others + xg - 1) / xg);
    while (others && xs < 3 && (vs * nv + (xs + 1) * xg) * KBLK <= room) ++xs;
    while (vs < MAX_VS && ((vs + 1) * nv + xs * xg) * KBLK <= room) ++vs;
    while (others && xs < MAX_XS && (vs * nv + (xs + 1) * xg) * KBLK <= room) ++xs;
    *L = Layout{nkb, chunks, nv, vs, xs, xg, nkb * QBLK + (vs * nv + xs * xg) * KBLK + (int)sizeof(Bars) + 1024,
                nv <= 2 ? 256 : 512, q_rows};
    return true;
  }
  return false;
}

}  // namespace

// Whether llm_attention_latent takes these sizes: returns the number of CTAs that share a group of
// 128 flat rows (parts of the value channels), or 0.  page_size: a multiple of 64, or 8, 16 or
// 32 positions.
LLM_EXPORT int llm_attention_latent_ok(int kd, int vdim, int page_size) {
  Layout L;
  if (kd <= 0 || kd % 8 || vdim <= 0 || vdim > kd) return 0;
  return page_size >= 8 && (page_size < KT ? KT % page_size == 0 : page_size % KT == 0) && layout_for(kd, vdim, ROWS, &L) ? L.chunks : 0;
}

// q [flat_rows][kd] and out [flat_rows][vdim] bfloat16, flat row = token * H + head; k_cache: this
// layer call's plane of key rows of page 0, page_stride elements from page to page, n_pages pages.
// items: device n_items x (first flat row, up to 128 flat rows, request slot, 0), all of one request
// each and consecutive; null: every token is a request of its own (n_items = flat_rows / H tokens).
// splits > 1: the keys of every row are cut into that many parts, part_o float32 [flat_rows][splits][vdim]
// and part_ml float32 [flat_rows][splits][2 x what llm_attention_latent_ok returns] take them, and the merge kernel follows.  sink: float32 [H]
// or null.  window: see first_key.
LLM_EXPORT int llm_attention_latent(const void* q, void* out, int flat_rows, int H, int kd, int vdim,
                                    const void* k_cache, long long page_stride, long long n_pages,
                                    const int* block_table, int table_stride, const int* items, int n_items,
                                    const int* row_pos, const int* row_slot, int page_size, float scale, int window,
                                    int splits, float* part_o, float* part_ml, const float* sink, int* status,
                                    cudaStream_t stream) {
  if (n_items <= 0 || flat_rows <= 0) return 0;
  if (H <= 0 || splits < 1 || splits > 1024 || (splits > 1 && (!part_o || !part_ml))) return LLM_ERR_ARGUMENT;
  if (!llm_attention_latent_ok(kd, vdim, page_size)) return LLM_ERR_UNSUPPORTED;
  if (((uintptr_t)q | (uintptr_t)out | (uintptr_t)k_cache | (uintptr_t)part_o) & 15) return LLM_ERR_UNSUPPORTED;
  if (page_stride % kd) return LLM_ERR_UNSUPPORTED;
  const long long rows_per_page = page_stride / kd;
  const long long key_rows = (n_pages - 1) * rows_per_page + page_size;
  if (n_pages <= 0 || key_rows >= (1LL << 31)) return LLM_ERR_UNSUPPORTED;
  Layout L;
  if (!layout_for(kd, vdim, ROWS, &L)) return LLM_ERR_UNSUPPORTED;
  {      // (the part of the value channels a CTA takes stays that of full groups of rows)
    const int q_rows = items || H >= ROWS ? ROWS : (H + 7) / 8 * 8;
    Layout M;
    if (layout_for(kd, vdim, q_rows, &M) && M.chunks == L.chunks) L = M;
  }
  CUtensorMap mq, mk;
  if (!llm_tensor_map(q, flat_rows, kd, kd, L.q_rows, 64, 0, &mq)) return LLM_ERR_UNSUPPORTED;
  if (!llm_tensor_map(k_cache, key_rows, kd, kd, page_size < KT ? page_size : KT, 64, 0, &mk)) return LLM_ERR_UNSUPPORTED;
  LatentArgs a;
  a.block_table = block_table, a.table_stride = table_stride, a.items = items;
  a.per_row = (H + ROWS - 1) / ROWS;
  a.q_rows = L.q_rows;
  a.row_pos = row_pos, a.row_slot = row_slot, a.rows_per_page = rows_per_page;
  a.H = H, a.page_size = page_size, a.kd_blocks = L.kd_blocks, a.vdim = vdim, a.v_blocks = L.v_blocks;
  a.chunks = L.chunks, a.vs = L.vs, a.xs = L.xs, a.xg = L.xg, a.tmem_cols = L.tmem_cols;
  a.scale_log2 = scale * 1.4426950408889634f, a.window = window, a.splits = splits;
  a.out = (bf16*)out, a.part_o = part_o, a.part_ml = part_ml, a.sink = sink, a.status = status;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(attention_latent_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_LIMIT);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const long long groups = items ? n_items : (long long)n_items * a.per_row;
  if (groups * L.chunks > 0x7fffffffLL) return LLM_ERR_UNSUPPORTED;
  int rc = launch_pdl(attention_latent_kernel, dim3((unsigned)(groups * L.chunks), splits), dim3(224), L.smem, stream, mq,
                      mk, a);
  if (rc || splits == 1) return rc;
  return launch_pdl(attention_latent_merge_kernel, dim3(flat_rows, L.chunks), dim3(128), splits * sizeof(float), stream,
                    (const float*)part_o, (const float*)part_ml, (bf16*)out, H, vdim, splits, L.v_blocks * 64, sink);
}
