// Causal attention of prompt portions over the paged KV cache on tcgen05 / TMEM (bf16).
//
// A portion is a run of consecutive tokens of one sequence whose keys and values are already in the
// cache (ft_qkv_finish / ft_qkv_head_finish / ft_kv_append); query token at position p sees keys 0 .. p,
// the last `window` of them, or those of its own chunk, which lie in pages named by the block table.  An item starts at
// the key block of its first token's first visible key.  A bias that grows with the distance (a slope per head) may be taken off the scores.  A step holds any number of portions of any lengths, so the work comes as a
// list of items: up to 2 * tpt consecutive tokens of one sequence, with all query heads of a KV group
// packed into the rows of the tile (row r = token r / group, head r % group; tpt = 128 / group tokens per
// 128-row tile).  Packing the group means that K and V are read once per group instead of once per head
// and that a portion of a few tokens still fills the tile.
//
// One CTA per (item, KV head), 384 threads, the structure of the two-tile kernel in attn_fwd.cu:
//   warp 0      producer: Q of both tiles once (one TMA box of [tpt tokens, group heads, 64] per chunk),
//               then 128-key K and V blocks, one TMA box per page and 64-wide chunk: lane i looks up and
//               loads page i of the block.  Rows of a page past the sequence's last token hold finite
//               values of other tokens; the mask takes their probability to zero.
//   warp 1      MMA issuer, alternating between the tiles: O_i += P_i V, then S_i = Q_i K_next^T
//   warp 2      TMEM allocator
//   warps 4-11  softmax groups of the two tiles (thread = query row), P written back over S in TMEM
// The epilogue adds the head's sink to the row sum, divides by it, multiplies by the output gate (per head
// or per element) and stores bf16.  Head sizes are multiples of 16 up to 128 and may differ between keys and values: the
// tensor maps end at the head's size, so the columns up to the tile's 64 or 128 are filled with zeros.
// Pooled blocks ahead of a window come first: tiles of 128 means, whose rows lie anywhere in the pooled pages, four to a
// TMA gather.
// All waits are bounded and report through the device status word.
#include "attn_row.cuh"
#include "ft_host.h"

namespace ft {

constexpr int PP_THREADS = 384;
constexpr int PP_KV_STAGES = 2;

template <int HD, int VD>
struct PpCfg {
  static constexpr int Q_BYTES = ATT_BM * HD * 2;   // one Q tile
  static constexpr int K_BYTES = ATT_BN * HD * 2;
  static constexpr int V_BYTES = ATT_BN * VD * 2;
  static constexpr int OFF_K = 2 * Q_BYTES;
  static constexpr int OFF_V = OFF_K + PP_KV_STAGES * K_BYTES;
  static constexpr int OFF_BAR = OFF_V + PP_KV_STAGES * V_BYTES;
  static constexpr int SMEM_BYTES = OFF_BAR + 256 + 1024;
  static constexpr int TMEM_COLS = 512;
  static constexpr int S_COL = 0;       // S_i at S_COL + i * 128; P_i aliases its first 64 columns
  static constexpr int O_COL = 256;     // O_i at O_COL + i * 128
};

struct PpParams {
  const int* items;         // [n_items, 4]: sequence slot, first query row, tokens, position of the first token
  const int* block_table;
  HeadGate gate;            // bf16
  const float* sink;
  __nv_bfloat16* out;
  const float* slopes;
  long long ldo;
  KeyRange range;
  PooledKeys pooled;
  int Hkv, group, tpt, D, Dv;
  int block_size, rows_per_box, boxes, max_blocks, num_blocks;
  float scale_log2, out_scale;
  int* status;
};

// What an instance can do beside plain causal attention (it costs registers that the plain kernel does not have to spare):
// PP_EXTRAS a window, chunks, sinks or a gate per element; PP_BIAS the distance bias as well; PP_POOL what PP_EXTRAS can, and
// pooled blocks.
enum : int { PP_PLAIN = 0, PP_EXTRAS = 1, PP_BIAS = 2, PP_POOL = 3 };

template <int HD, int VD, int KIND>
__global__ void __launch_bounds__(PP_THREADS, 1)
paged_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                     const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmKp,
                     const __grid_constant__ CUtensorMap tmVp, const PpParams p) {
  using Cfg = PpCfg<HD, VD>;
  constexpr bool EXTRAS = KIND != PP_PLAIN;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  const uint32_t sbase = smem_u32(smem);
  const uint32_t sQ = sbase, sK = sbase + Cfg::OFF_K, sV = sbase + Cfg::OFF_V;
  const uint32_t bar0 = sbase + Cfg::OFF_BAR;
  enum { Q_FULL = 0, K_FULL = 2, K_EMPTY = 4, V_FULL = 6, V_EMPTY = 8, S_FULL = 10, P_FULL = 12,
         O_DONE = 14, NBARS = 16 };
  auto bar = [&](int i) { return bar0 + 8u * i; };
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + Cfg::OFF_BAR + 8 * NBARS);
  volatile int* abort_word = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kvh = blockIdx.y;
  const int slot = p.items[4 * blockIdx.x], row0 = p.items[4 * blockIdx.x + 1];
  const int n_tok = p.items[4 * blockIdx.x + 2], pos0 = p.items[4 * blockIdx.x + 3];
  // tokens and key blocks of each tile
  int nt[2], nb[2];
  // blocks of pooled means, which the item's last token sees, then blocks of keys: number n_pool of this item is key block j0
  const int pool_seen = KIND == PP_POOL ? p.pooled.count(p.range.first_visible(pos0 + n_tok)) : 0;
  const int n_pool = (pool_seen + ATT_BN - 1) / ATT_BN;
  const int j0 = EXTRAS ? p.range.first_visible(pos0 + 1) / ATT_BN : 0;
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    nt[i] = min(max(n_tok - i * p.tpt, 0), p.tpt);
    nb[i] = nt[i] > 0 ? (pos0 + i * p.tpt + nt[i] + ATT_BN - 1) / ATT_BN - j0 + n_pool : 0;
  }
  const int n_blocks = max(nb[0], nb[1]);

  if (threadIdx.x == 0) {
    *abort_word = 0;
    for (int i = 0; i < 2; ++i) {
      mbar_init(bar(Q_FULL + i), 1);
      mbar_init(bar(K_FULL + i), 1);
      mbar_init(bar(K_EMPTY + i), 1);
      mbar_init(bar(V_FULL + i), 1);
      mbar_init(bar(V_EMPTY + i), 1);
      mbar_init(bar(S_FULL + i), 1);
      mbar_init(bar(P_FULL + i), 4);  // one arrival per softmax warp of the tile
      mbar_init(bar(O_DONE + i), 1);
    }
    fence_mbar_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
    if (KIND == PP_POOL) {
      tma_prefetch_desc(&tmKp);
      tma_prefetch_desc(&tmVp);
    }
  }
  if (warp == 2) {
    tmem_alloc(smem_u32(tmem_slot), Cfg::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    // ------------------------------------------------------------------ producer (whole warp)
    if (n_blocks > 0) {
      if (lane == 0) {
        const uint32_t q_bytes = static_cast<uint32_t>(p.tpt * p.group * 128 * (HD / 64));   // boxes count in full
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          if (nb[i] == 0) continue;
          mbar_expect_tx(bar(Q_FULL + i), q_bytes);
#pragma unroll
          for (int c = 0; c < HD / 64; ++c)
            tma_load_3d(sQ + i * Cfg::Q_BYTES + c * (ATT_BM * 128), &tmQ, bar(Q_FULL + i), c * 64, kvh * p.group,
                        row0 + i * p.tpt);
        }
      }
      const int* bt = p.block_table + static_cast<long long>(slot) * p.max_blocks;
      // box `lane` of key block j: rows_per_box keys of one page, as a row of the [num_blocks * block_size] axis
      auto page_row = [&](int j) {
        const int key = (j0 + j - n_pool) * ATT_BN + lane * p.rows_per_box;
        const int page = min(key / p.block_size, p.max_blocks - 1);
        const int blk = min(max(lane < p.boxes ? __ldg(bt + page) : 0, 0), p.num_blocks - 1);
        return blk * p.block_size + key % p.block_size;
      };
      // pooled block 4 * lane + i of tile j, as a row of the [num_blocks * per_page * Hkv] axis; past the last one: that one again
      auto pool_row = [&](int j, int i) {
        const int b = min(j * ATT_BN + lane * 4 + i, pool_seen - 1);
        return static_cast<int>(p.pooled.row(b, bt, p.block_size, p.max_blocks, p.num_blocks)) * p.Hkv + kvh;
      };
      int row = n_pool > 0 ? 0 : page_row(0);
      bool ok = true;
      for (int j = 0; j < n_blocks; ++j) {
        const int st = j & 1;
        const uint32_t par = ((j >> 1) & 1) ^ 1u;
        const int next_row = j + 1 < n_blocks && j + 1 >= n_pool ? page_row(j + 1) : 0;
        const bool is_pool = KIND == PP_POOL && j < n_pool;
        int pr[4];
        if (is_pool) {
#pragma unroll
          for (int i = 0; i < 4; ++i) pr[i] = pool_row(j, i);
        }
        ok = mbar_wait(bar(K_EMPTY + st), par, abort_word, FT_ERR_TIMEOUT_PRODUCER);
        if (!__all_sync(0xffffffffu, ok)) break;
        if (lane == 0) mbar_expect_tx(bar(K_FULL + st), Cfg::K_BYTES);
        __syncwarp();
        if (is_pool) {
#pragma unroll
          for (int c = 0; c < HD / 64; ++c)
            tma_gather4_2d(sK + st * Cfg::K_BYTES + c * (ATT_BN * 128) + lane * 512, &tmKp, bar(K_FULL + st), c * 64, pr[0], pr[1], pr[2], pr[3]);
        } else if (lane < p.boxes) {
#pragma unroll
          for (int c = 0; c < HD / 64; ++c)
            tma_load_3d(sK + st * Cfg::K_BYTES + c * (ATT_BN * 128) + lane * p.rows_per_box * 128, &tmK, bar(K_FULL + st),
                        c * 64, kvh, row);
        }
        ok = mbar_wait(bar(V_EMPTY + st), par, abort_word, FT_ERR_TIMEOUT_PRODUCER);
        if (!__all_sync(0xffffffffu, ok)) break;
        if (lane == 0) mbar_expect_tx(bar(V_FULL + st), Cfg::V_BYTES);
        __syncwarp();
        if (is_pool) {
#pragma unroll
          for (int c = 0; c < VD / 64; ++c)
            tma_gather4_2d(sV + st * Cfg::V_BYTES + c * (ATT_BN * 128) + lane * 512, &tmVp, bar(V_FULL + st), c * 64, pr[0], pr[1], pr[2], pr[3]);
        } else if (lane < p.boxes) {
#pragma unroll
          for (int c = 0; c < VD / 64; ++c)
            tma_load_3d(sV + st * Cfg::V_BYTES + c * (ATT_BN * 128) + lane * p.rows_per_box * 128, &tmV, bar(V_FULL + st),
                        c * 64, kvh, row);
        }
        row = next_row;
      }
      if (*abort_word) {   // let copies in flight land before the CTA leaves
        const unsigned long long t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0 && n_blocks > 0) {
      constexpr uint32_t idesc_qk = make_idesc_f16(ATT_BM, ATT_BN, 1, 0, 0);
      constexpr uint32_t idesc_pv = make_idesc_f16(ATT_BM, VD, 1, 0, 1);
      const int ksteps = p.D / 16;                 // the columns past the head size are zeros
      bool ok = true;
      // S_i = Q_i K_j^T into the tile's S columns
      auto issue_qk = [&](int i, int j) {
        const uint32_t kbase = sK + (j & 1) * Cfg::K_BYTES;
        const uint32_t qbase = sQ + i * Cfg::Q_BYTES;
        const uint32_t d = tmem_base + Cfg::S_COL + i * ATT_BN;
#pragma unroll
        for (int kk = 0; kk < HD / 16; ++kk) {
          if (kk < ksteps) {
            const uint32_t off = (kk >> 2) * (ATT_BM * 128) + (kk & 3) * 32;
            umma_f16_ss(d, make_smem_desc_sw128(qbase + off, 16, 1024),
                        make_smem_desc_sw128(kbase + off, 16, 1024), idesc_qk, kk > 0 ? 1u : 0u);
          }
        }
        umma_commit(bar(S_FULL + i));
      };
      // O_i += P_i V_j with P_i read from tensor memory
      auto issue_pv = [&](int i, int j) {
        const uint32_t vbase = sV + (j & 1) * Cfg::V_BYTES;
        const uint32_t d = tmem_base + Cfg::O_COL + i * 128;
        const uint32_t a = tmem_base + Cfg::S_COL + i * ATT_BN;
#pragma unroll
        for (int kk = 0; kk < ATT_BN / 16; ++kk)
          umma_f16_ts(d, a + kk * 8, make_smem_desc_sw128(vbase + kk * 2048, ATT_BN * 128, 1024), idesc_pv,
                      (j > 0 || kk > 0) ? 1u : 0u);
        umma_commit(bar(O_DONE + i));
      };
      // block 0 scores of both tiles
      ok = mbar_wait(bar(K_FULL + 0), 0, abort_word, FT_ERR_TIMEOUT_MMA);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        if (nb[i] == 0 || !ok) continue;
        ok = mbar_wait(bar(Q_FULL + i), 0, abort_word, FT_ERR_TIMEOUT_MMA);
        if (!ok) break;
        tc_fence_after();
        issue_qk(i, 0);
      }
      if (ok) umma_commit(bar(K_EMPTY + 0));  // stage 0 is free once the block-0 scores are done
      for (int j = 0; j < n_blocks && ok; ++j) {
        const int st = j & 1;
        const bool has_next = j + 1 < n_blocks;
        if (has_next) {
          ok = mbar_wait(bar(K_FULL + (st ^ 1)), ((j + 1) >> 1) & 1, abort_word, FT_ERR_TIMEOUT_MMA);
          if (!ok) break;
        }
        ok = mbar_wait(bar(V_FULL + st), (j >> 1) & 1, abort_word, FT_ERR_TIMEOUT_MMA);
        if (!ok) break;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          if (j < nb[i]) {
            ok = mbar_wait(bar(P_FULL + i), j & 1, abort_word, FT_ERR_TIMEOUT_MMA);
            if (!ok) break;
            tc_fence_after();
            issue_pv(i, j);
          }
          if (j + 1 < nb[i]) {
            tc_fence_after();
            issue_qk(i, j + 1);
          }
        }
        if (!ok) break;
        // every MMA that reads this V stage (and the K stage of block j + 1) has been issued
        umma_commit(bar(V_EMPTY + st));
        if (has_next) umma_commit(bar(K_EMPTY + (st ^ 1)));
      }
    }
  } else if (warp >= 4) {
    // ------------------------------------------------------------------ softmax groups
    const int ti = (warp - 4) >> 2;  // tile of this warpgroup
    const int ew = warp & 3;         // TMEM lane quarter
    const int r = ew * 32 + lane;
    const int tok = r / p.group, head = r - tok * p.group;
    const int my_nb = nb[ti];
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(ew * 32) << 16);
    const uint32_t s_addr = lane_addr + Cfg::S_COL + ti * ATT_BN;
    const uint32_t o_addr = lane_addr + Cfg::O_COL + ti * 128;
    float m_ref = -INFINITY;  // reference maximum the stored P and O are relative to
    float l = 0.f;
    bool ok = true;
    const int tile_pos = pos0 + ti * p.tpt;
    const int limit = tile_pos + tok;                              // last visible key
    const int warp_limit = tile_pos + (ew * 32) / p.group;         // of this warp's first row
    const int pool_limit = KIND == PP_POOL ? p.pooled.count(p.range.first_visible(limit + 1)) - 1 : 0;       // last visible pooled block
    const int warp_pool_limit = KIND == PP_POOL ? p.pooled.count(p.range.first_visible(warp_limit + 1)) - 1 : 0;
    float slope = 0.f;                                             // in powers of two per position
    if constexpr (KIND == PP_BIAS)
      if (p.slopes) slope = p.slopes[min(kvh * p.group + head, p.Hkv * p.group - 1)] * ATT_LOG2E;
    const float row_scale = KIND == PP_BIAS ? 1.f : p.scale_log2;  // what a score is still to be multiplied by
    for (int j = 0; j < my_nb && ok; ++j) {
      if (!mbar_wait(bar(S_FULL + ti), j & 1, abort_word, FT_ERR_TIMEOUT_EPILOGUE)) { ok = false; break; }
      tc_fence_after();
      f32x2 sp[ATT_BN / 2];
      att2_load_row(s_addr, sp);
      const bool is_pool = KIND == PP_POOL && j < n_pool;
      const int kv0 = is_pool ? j * ATT_BN : (j0 + j - n_pool) * ATT_BN;
      if constexpr (KIND == PP_BIAS) {                             // score * scale - slope * (limit - key)
        const f32x2 sc = f2_pack(p.scale_log2, p.scale_log2), two = f2_pack(2.f * slope, 2.f * slope);
        const float b0 = slope * static_cast<float>(kv0 - limit);
        f32x2 bias = f2_pack(b0, b0 + slope);
#pragma unroll
        for (int i = 0; i < ATT_BN / 2; ++i) {
          sp[i] = f2_fma(sp[i], sc, f2_fma(two, f2_pack(static_cast<float>(i), static_cast<float>(i)), bias));
        }
      }
      const int last_seen = is_pool ? pool_limit : limit;
      if (kv0 + ATT_BN - 1 > (is_pool ? warp_pool_limit : warp_limit)) att2_mask_row(sp, kv0, last_seen);   // warp-uniform branches
      // no row of the warp is more than 31 positions past its first; a row may see nothing of its first blocks
      if (EXTRAS && !is_pool && kv0 < p.range.first_visible(warp_limit + 32)) att2_mask_ahead(sp, kv0, p.range.first_visible(limit + 1));
      const float mx = att2_row_max(sp) * row_scale;     // scale > 0, so the maximum commutes with it
      float alpha = 1.f;
      if (mx > m_ref + ATT2_RESCALE_THRESHOLD) {
        alpha = fast_exp2(m_ref - mx);  // m_ref = -inf on the first block -> 0
        m_ref = mx;
      }
      const float m_use = (m_ref == -INFINITY) ? 0.f : m_ref;
      uint32_t pk[ATT_BN / 2];
      const float rowsum = att2_exp_row(sp, row_scale, -m_use, pk);
      l = l * alpha + rowsum;
      if (j > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
        // O of the previous blocks is relative to the old reference: bring it to the new one
        if (!mbar_wait(bar(O_DONE + ti), (j - 1) & 1, abort_word, FT_ERR_TIMEOUT_EPILOGUE)) { ok = false; break; }
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < VD / 32; ++c) {
          uint32_t t[32];
          tmem_ld_32x32(o_addr + c * 32, t);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) t[i] = __float_as_uint(__uint_as_float(t[i]) * alpha);
          tmem_st_32x32(o_addr + c * 32, t);
        }
      }
      // P (bf16, two keys per 32-bit column) over the first 64 columns of this tile's S
      {
        uint32_t(&lo)[32] = *reinterpret_cast<uint32_t(*)[32]>(&pk[0]);
        uint32_t(&hi)[32] = *reinterpret_cast<uint32_t(*)[32]>(&pk[32]);
        tmem_st_32x32(s_addr, lo);
        tmem_st_32x32(s_addr + 32, hi);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar(P_FULL + ti));
    }
    if (ok && my_nb > 0) {
      ok = mbar_wait(bar(O_DONE + ti), (my_nb - 1) & 1, abort_word, FT_ERR_TIMEOUT_EPILOGUE);
      tc_fence_after();
    }
    if (ok && my_nb > 0) {
      const bool row_ok = tok < nt[ti];
      const long long row = static_cast<long long>(row0) + ti * p.tpt + tok;
      const int hq = kvh * p.group + head;
      float m = m_ref, num = 1.f;
      if constexpr (EXTRAS) sink_join(p.sink, min(hq, p.Hkv * p.group - 1), m, l, num);
      float inv_l = l > 0.f ? num / l * p.out_scale : 0.f;
      if (p.gate.g && row_ok && p.gate.elem == 0) inv_l *= head_gate_bf16(p.gate, static_cast<int>(row), hq, 0);
      const bool elem_gate = EXTRAS && p.gate.g && p.gate.elem != 0;
      __nv_bfloat16* orow = p.out + row * p.ldo + static_cast<long long>(hq) * p.Dv;
#pragma unroll
      for (int c = 0; c < VD / 32; ++c) {
        uint32_t t[32];
        tmem_ld_32x32(o_addr + c * 32, t);
        tmem_ld_wait();
        if (row_ok) {
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            const int d = c * 32 + g * 8;
            if (d >= p.Dv) continue;
            float f[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(t[g * 8 + e]) * inv_l;
            if (elem_gate) {
              const uint4 z = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.gate.g) +
                                                              p.gate.at(static_cast<int>(row), hq, d));
              const float2 z0 = unpack_bf16x2(z.x), z1 = unpack_bf16x2(z.y), z2 = unpack_bf16x2(z.z), z3 = unpack_bf16x2(z.w);
              f[0] *= gate_value_bf16(z0.x); f[1] *= gate_value_bf16(z0.y); f[2] *= gate_value_bf16(z1.x); f[3] *= gate_value_bf16(z1.y);
              f[4] *= gate_value_bf16(z2.x); f[5] *= gate_value_bf16(z2.y); f[6] *= gate_value_bf16(z3.x); f[7] *= gate_value_bf16(z3.y);
            }
            uint4 o;
            o.x = pack_bf16x2(f[0], f[1]);
            o.y = pack_bf16x2(f[2], f[3]);
            o.z = pack_bf16x2(f[4], f[5]);
            o.w = pack_bf16x2(f[6], f[7]);
            *reinterpret_cast<uint4*>(orow + c * 32 + g * 8) = o;
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 2) {
    tc_fence_after();
    tmem_dealloc(tmem_base, Cfg::TMEM_COLS);
  }
  if (threadIdx.x == 0 && *abort_word != 0 && p.status) atomicCAS(p.status, 0, *abort_word);
}

template <int HD, int VD, int KIND>
static int launch_prefill(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const CUtensorMap& tkp, const CUtensorMap& tvp,
                                const PpParams& p, int n_items, int device, cudaStream_t stream) {
  using Cfg = PpCfg<HD, VD>;
  auto kern = paged_prefill_kernel<HD, VD, KIND>;
  static bool attr_set[64] = {false};
  if (!attr_set[device]) {
    FT_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM_BYTES));
    attr_set[device] = true;
  }
  kern<<<dim3(n_items, p.Hkv), PP_THREADS, Cfg::SMEM_BYTES, stream>>>(tq, tk, tv, tkp, tvp, p);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

template <int HD, int VD>
static int launch_paged_prefill(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const CUtensorMap& tkp, const CUtensorMap& tvp,
                                const PpParams& p, int n_items, int device, cudaStream_t stream) {
  if (p.pooled.pool > 0) return launch_prefill<HD, VD, PP_POOL>(tq, tk, tv, tkp, tvp, p, n_items, device, stream);
  if (p.slopes) return launch_prefill<HD, VD, PP_BIAS>(tq, tk, tv, tkp, tvp, p, n_items, device, stream);
  const bool extras = p.range.window > 0 || p.range.chunk > 0 || p.sink || (p.gate.g && p.gate.elem != 0);
  return extras ? launch_prefill<HD, VD, PP_EXTRAS>(tq, tk, tv, tkp, tvp, p, n_items, device, stream)
                : launch_prefill<HD, VD, PP_PLAIN>(tq, tk, tv, tkp, tvp, p, n_items, device, stream);
}

}  // namespace ft

// Query tokens per 128-row tile when `group` query heads share a KV head; a work item holds up to twice as many.
FT_API int ft_paged_prefill_tile(int group) { return group > 0 && group <= ft::ATT_BM ? ft::ATT_BM / group : 0; }

// Attention of prompt portions (see the top of this file).  q: [rows, Hq, D] (row stride ldq), out: [rows,
// Hq, Dv] (row stride ldo); window, chunk, pool, slopes, sink, gate and out_scale as in ft_paged_decode (a gate per element has unit element stride
// and 16-byte aligned heads).  items: int32 [n_items, 4] on the
// device: slot, first query row, number of tokens (<= 2 * ft_paged_prefill_tile), position of the first token;
// keys 0 .. position of a token must be in the cache.  Page sizes: a divisor of 128 of at least 8, or a
// multiple of 128.  scale > 0.
FT_API int ft_paged_prefill(const void* q, const void* k_cache, const void* v_cache, const int* block_table, const int* items,
                            const void* gate, const float* sink, void* out, int n_items, int rows, int Hq, int Hkv, int D,
                            int Dv, long long ldq, long long ldg, int gate_head, int gate_elem, long long ldo, int block_size,
                            int max_blocks, int num_blocks, float scale, int window, int chunk, const void* k_pool, const void* v_pool, int pool,
                            const float* slopes, float out_scale, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  using namespace ft;
  FT_REQUIRE(q && k_cache && v_cache && block_table && items && out, "ft_paged_prefill: null pointer");
  FT_REQUIRE(rows > 0 && Hq > 0 && Hkv > 0 && Hq % Hkv == 0 && Hq / Hkv <= ATT_BM && max_blocks > 0 && num_blocks > 0, "ft_paged_prefill: bad shape");
  FT_REQUIRE(D >= 16 && D <= 128 && D % 16 == 0 && Dv >= 16 && Dv <= 128 && Dv % 16 == 0,
             "ft_paged_prefill: head sizes %d / %d must be multiples of 16 up to 128", D, Dv);
  FT_REQUIRE(block_size >= 8 && (128 % block_size == 0 || block_size % 128 == 0), "ft_paged_prefill: page size %d", block_size);
  FT_REQUIRE(static_cast<long long>(num_blocks) * block_size < (1ll << 31), "ft_paged_prefill: the cache is too large");
  FT_REQUIRE(ldq % 8 == 0 && ldo % 8 == 0 && scale > 0.f && ldq >= static_cast<long long>(Hq) * D,
             "ft_paged_prefill: strides must be multiples of 8 elements and the scale positive");
  FT_REQUIRE(((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) |
               reinterpret_cast<uintptr_t>(out)) & 15) == 0, "ft_paged_prefill: pointers must be 16-byte aligned");
  FT_REQUIRE(window >= 0 && chunk >= 0 && (!gate || gate_elem == 0 || (gate_elem == 1 && gate_head % 8 == 0 && ldg % 8 == 0 &&
                                                         (reinterpret_cast<uintptr_t>(gate) & 15) == 0)),
             "ft_paged_prefill: the window is negative or the gate's elements are not packed and aligned");
  FT_REQUIRE(pool == 0 || (pool > 0 && window > 0 && !chunk && !slopes && k_pool && v_pool &&
                           ((reinterpret_cast<uintptr_t>(k_pool) | reinterpret_cast<uintptr_t>(v_pool)) & 15) == 0), "ft_paged_prefill: blocks of %d keys", pool);
  if (n_items <= 0) return FT_E_OK;
  PpParams p;
  p.items = items; p.block_table = block_table; p.gate = HeadGate{gate, ldg, gate_head, gate_elem};
  p.sink = sink; p.slopes = slopes; p.range = KeyRange{window, chunk}; p.pooled = pooled_keys(k_pool, v_pool, pool, block_size); p.out_scale = out_scale;
  p.out = static_cast<__nv_bfloat16*>(out); p.ldo = ldo;
  p.Hkv = Hkv; p.group = Hq / Hkv; p.tpt = ATT_BM / p.group; p.D = D; p.Dv = Dv;
  p.block_size = block_size;
  p.rows_per_box = block_size < ATT_BN ? block_size : ATT_BN;
  p.boxes = ATT_BN / p.rows_per_box;
  p.max_blocks = max_blocks; p.num_blocks = num_blocks;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.status = device_status_word(device);
  CUtensorMap tq, tk, tv;
  int rc = make_tmap_3d(&tq, q, 2, D, Hq, rows, static_cast<uint64_t>(D) * 2, static_cast<uint64_t>(ldq) * 2, 64, p.group, p.tpt, 3);
  if (rc) return rc;
  const uint64_t n_rows = static_cast<uint64_t>(num_blocks) * block_size;
  rc = make_tmap_3d(&tk, k_cache, 2, D, Hkv, n_rows, static_cast<uint64_t>(D) * 2, static_cast<uint64_t>(Hkv) * D * 2, 64, 1,
                    p.rows_per_box, 3);
  if (rc) return rc;
  rc = make_tmap_3d(&tv, v_cache, 2, Dv, Hkv, n_rows, static_cast<uint64_t>(Dv) * 2, static_cast<uint64_t>(Hkv) * Dv * 2, 64, 1,
                    p.rows_per_box, 3);
  if (rc) return rc;
  CUtensorMap tkp = tk, tvp = tv;
  if (pool > 0) {
    const uint64_t pool_rows = static_cast<uint64_t>(num_blocks) * p.pooled.per_page * Hkv;
    FT_REQUIRE(pool_rows < (1ull << 31), "ft_paged_prefill: the cache is too large");
    if (int rc2 = make_tmap_2d(&tkp, k_pool, 2, D, pool_rows, static_cast<uint64_t>(D) * 2, 64, 1, 3)) return rc2;
    if (int rc2 = make_tmap_2d(&tvp, v_pool, 2, Dv, pool_rows, static_cast<uint64_t>(Dv) * 2, 64, 1, 3)) return rc2;
  }
  if (D > 64)
    return Dv > 64 ? launch_paged_prefill<128, 128>(tq, tk, tv, tkp, tvp, p, n_items, device, stream)
                   : launch_paged_prefill<128, 64>(tq, tk, tv, tkp, tvp, p, n_items, device, stream);
  return Dv > 64 ? launch_paged_prefill<64, 128>(tq, tk, tv, tkp, tvp, p, n_items, device, stream)
                 : launch_paged_prefill<64, 64>(tq, tk, tv, tkp, tvp, p, n_items, device, stream);
}
