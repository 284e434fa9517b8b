// Latent attention over the paged cache: a token's cached row is its latent c (of `rank` elements) followed by one rotated
// key part that all heads share; keys and values of a head are linear in c.
//
//   ft_latent_finish   everything between the packed projection [ q heads | latent | rotated key part | .. ] and the
//                      attention: RMS norm of the latent, rotation of the key part and of every head's rotated
//                      query part (neighbouring elements are pairs), the row into its cache page
//   ft_latent_decode   one query token per row, queries already in the latent space: all heads of a row attend to the cached
//                      rows themselves, o = softmax(scale * q . row) row[0 .. rank), split over the context (bf16)
//   ft_latent_gather   the cached rows of portions' contexts, contiguous: the operand from which the keys and values of
//                      a prompt portion are formed
//
// Decoding reads every cached row once for up to 32 heads.  A CTA owns (context split, group of heads, row) and walks the keys in
// tiles of 128, the layout of paged_decode_tc_kernel (paged_attn.cu) with the values inside the keys:
//     S^T[key, head]  = sum over 64-column pieces of the tile  (M = 128 keys, N = heads)
//     O^T[d, head]   += tile[:, d]^T P^T                       (one MMA chain per 128 latent columns)
// A tile of 576 columns takes 144 KB, so there is one; its pieces are ring slots of their own: a piece is loaded again as soon as
// the last product that reads it has finished, while the others are still in use.
//   warp 0  producer: one TMA box per page and piece     warp 1  MMA issuer     warp 2  TMEM allocator
//   warps 4-   softmax (thread = key) and epilogue (thread = latent column), four warps for every 16 heads
// All waits are bounded and report through the device status word.
#include <initializer_list>

#include "row_vec.cuh"

namespace ft {

constexpr int LF_ROWS = 4;        // rows of a block
constexpr int LF_MAX_THREADS = 32 * LF_ROWS + 256;
constexpr int LF_KEEP = 3;        // vectors of eight elements of the latent that a lane keeps

struct LatentFinishParams {
  void* packed;             // [rows, ld]
  void* q_lat;              // [n_lat, H, rank_pad + rot_pad]: rows 0 .. n_lat - 1 put their rotated query parts here, behind the latent part
  const int* pos;
  const int* slots;
  const int* block_table;
  void* cache;              // [num_blocks, block_size, rank_pad + rot_pad]
  const float* weight;      // [rank_pad]
  const float2* table;      // [positions, half]
  long long ld;
  int rows, n_lat, H, q_off, q_head, q_rot, c_off, rank_pad, rank, rot_pad, half, positions;
  float eps;
  int block_size, max_blocks, num_blocks;
};

// Eight elements d .. d + 7 of a rotated part: pairs (2i, 2i + 1), i < half, turn.
__device__ __forceinline__ void rotate8(float (&f)[8], int d, const float2* cs, int half) {
#pragma unroll
  for (int e = 0; e < 8; e += 2) {
    const int i = (d + e) / 2;
    if (i < half) {
      const float2 t = __ldg(cs + i);
      const float u = f[e], v = f[e + 1];
      f[e] = u * t.x - v * t.y;
      f[e + 1] = v * t.x + u * t.y;
    }
  }
}

// A block takes LF_ROWS rows: one warp each for their latents and key parts, the other threads their queries (a thread the same
// place of every row, all loads in flight together).
template <typename T>
__global__ void __launch_bounds__(LF_MAX_THREADS)
latent_finish_kernel(const LatentFinishParams p) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int width = p.rank_pad + p.rot_pad;
  const int row0 = blockIdx.x * LF_ROWS;
  auto angles = [&](int row) { return p.table + static_cast<long long>(min(p.pos[row], p.positions - 1)) * p.half; };
  if (warp < LF_ROWS) {
    const int row = row0 + warp;
    if (row >= p.rows) return;
    const T* c = static_cast<const T*>(p.packed) + static_cast<long long>(row) * p.ld + p.c_off;
    float kept[LF_KEEP][8];
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < LF_KEEP; ++k) {
      const int i = (k * 32 + lane) * 8;
      if (i < width) load8(c + i, kept[k]);
    }
    const int position = p.pos[row], page = position / p.block_size;
    const float2* cs = angles(row);
    const int blk = page < p.max_blocks ? p.block_table[static_cast<long long>(p.slots[row]) * p.max_blocks + page] : -1;
    if (blk < 0 || blk >= p.num_blocks) return;        // a row of no sequence
    T* dst = static_cast<T*>(p.cache) + (static_cast<long long>(blk) * p.block_size + position % p.block_size) * width;
#pragma unroll
    for (int k = 0; k < LF_KEEP; ++k)
      if ((k * 32 + lane) * 8 < p.rank_pad)
#pragma unroll
        for (int e = 0; e < 8; ++e) sum += kept[k][e] * kept[k][e];
    const int rest = (LF_KEEP * 32 + lane) * 8;        // wider rows are read twice
    for (int i = rest; i < p.rank_pad; i += 256) {
      float f[8];
      load8(c + i, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) sum += f[e] * f[e];
    }
    const float r = 1.f / sqrtf(warp_sum(sum) / static_cast<float>(p.rank) + p.eps);
    auto finish = [&](int i, float (&f)[8]) {
      if (i < p.rank_pad) {
        float w[8];
        load8(p.weight + i, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] *= r * w[e];
      } else {
        rotate8(f, i - p.rank_pad, cs, p.half);
      }
      store8(dst + i, f);
    };
#pragma unroll
    for (int k = 0; k < LF_KEEP; ++k) {
      const int i = (k * 32 + lane) * 8;
      if (i < width) finish(i, kept[k]);
    }
    for (int i = rest; i < width; i += 256) {
      float f[8];
      load8(c + i, f);
      finish(i, f);
    }
  } else {
    const int units = p.rot_pad / 8;
    for (int u = threadIdx.x - 32 * LF_ROWS; u < p.H * units; u += blockDim.x - 32 * LF_ROWS) {
      const int h = u / units, d = (u - h * units) * 8;
      float f[LF_ROWS][8];
      const float2* cs[LF_ROWS];
      T* q[LF_ROWS];
#pragma unroll
      for (int k = 0; k < LF_ROWS; ++k) {              // past the end: the last row again, not stored
        const int row = min(row0 + k, p.rows - 1);
        q[k] = static_cast<T*>(p.packed) + static_cast<long long>(row) * p.ld + p.q_off + static_cast<long long>(h) * p.q_head + p.q_rot + d;
        load8(q[k], f[k]);
        cs[k] = angles(row);
      }
#pragma unroll
      for (int k = 0; k < LF_ROWS; ++k) rotate8(f[k], d, cs[k], p.half);
#pragma unroll
      for (int k = 0; k < LF_ROWS; ++k) {
        const int row = row0 + k;
        if (row < p.rows)
          store8(row < p.n_lat ? static_cast<T*>(p.q_lat) + (static_cast<long long>(row) * p.H + h) * width + p.rank_pad + d : q[k], f[k]);
      }
    }
  }
}

// ---------------------------------------------------------------- decode
constexpr int LD_GROUP = 16;               // heads of a softmax group
constexpr int LD_TILE = 128;               // keys
constexpr int LD_PIECE = LD_TILE * 128;    // bytes of 64 columns
constexpr int LD_MAX_PIECES = 9;
constexpr float LD_RESCALE = 8.f;

template <int N>
struct LdCfg {
  static constexpr int GROUPS = N / LD_GROUP;
  static constexpr int THREADS = 128 + 128 * GROUPS;
  static constexpr int Q_PIECE = N * 128;
  static constexpr int P_BYTES = 2 * N * 128;             // two pieces of 64 keys
  static constexpr int OFF_Q = LD_MAX_PIECES * LD_PIECE;
  static constexpr int OFF_P = OFF_Q + LD_MAX_PIECES * Q_PIECE;
  static constexpr int OFF_RED = OFF_P + P_BYTES;         // per group [4 warps][16] floats, then [16] references
  static constexpr int OFF_BAR = OFF_RED + 5 * N * 4;
  static constexpr int SMEM_BYTES = OFF_BAR + 256 + 1024;
  static constexpr uint32_t TMEM_COLS = N * 5 <= 128 ? 128 : 256;
};

struct LatentDecodeParams {
  const __nv_bfloat16* q;    // [B, H, width]
  const int* block_table;
  const int* row_slot;
  const int* ctx_len;
  __nv_bfloat16* out;        // [B, H, rank] (row stride ldo)
  float* part_o;
  float* part_ml;
  long long ldo;
  int H, width, rank, pieces, v_pieces;      // v_pieces: 64-column pieces that the value products read (even)
  int block_size, rows_per_box, boxes, max_blocks, num_blocks, n_splits;
  float scale_log2;
  int* status;
};

template <int N>
__global__ void __launch_bounds__(LdCfg<N>::THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmC, const LatentDecodeParams p) {
  using Cfg = LdCfg<N>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const uint32_t sbase = smem_u32(smem);
  enum { FULL = 0, EMPTY = FULL + LD_MAX_PIECES, S_FULL = EMPTY + LD_MAX_PIECES, P_FULL, O_DONE, NBARS };
  const uint32_t bar0 = sbase + Cfg::OFF_BAR;
  auto bar = [&](int i) { return bar0 + 8u * i; };
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + Cfg::OFF_BAR + 8 * NBARS);
  volatile int* abort_word = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int split = blockIdx.x, h0 = blockIdx.y * N, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int heads = min(N, p.H - h0);
  const int len = min(p.ctx_len[b], p.max_blocks * p.block_size);
  const int tiles = (len + LD_TILE - 1) / LD_TILE, per_split = (tiles + p.n_splits - 1) / p.n_splits;
  const int tile_lo = split * per_split, n_tiles = max(0, min(tiles, tile_lo + per_split) - tile_lo);
  const int blocks = p.v_pieces / 2;         // 128-column blocks of the latent

  if (threadIdx.x == 0) {
    *abort_word = 0;
    for (int i = 0; i < LD_MAX_PIECES; ++i) {
      mbar_init(bar(FULL + i), 1);
      mbar_init(bar(EMPTY + i), 1);
    }
    mbar_init(bar(S_FULL), 1);
    mbar_init(bar(P_FULL), 4 * Cfg::GROUPS);
    mbar_init(bar(O_DONE), 1);
    fence_mbar_init();
    tma_prefetch_desc(&tmC);
  }
  if (warp == 2) {
    tmem_alloc(smem_u32(tmem_slot), Cfg::TMEM_COLS);
    tmem_relinquish();
  }
  // the queries as the B operand (rows past the heads and columns past the width zero)
  for (int i = threadIdx.x; i < N * LD_MAX_PIECES * 8; i += Cfg::THREADS) {
    const int h = i / (LD_MAX_PIECES * 8), u = i - h * (LD_MAX_PIECES * 8);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (h < heads && u * 8 < p.width) v = *reinterpret_cast<const uint4*>(p.q + (static_cast<long long>(b) * p.H + h0 + h) * p.width + u * 8);
    *reinterpret_cast<uint4*>(smem + Cfg::OFF_Q + (u >> 3) * Cfg::Q_PIECE + h * 128 + (((u & 7) ^ (h & 7)) << 4)) = v;
  }
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint32_t COL_S = 0, COL_O = N;       // O^T of block i at COL_O + i * N

  if (warp == 0) {
    // ------------------------------------------------------------------ producer (whole warp)
    const int* bt = p.block_table + static_cast<long long>(p.row_slot ? p.row_slot[b] : b) * p.max_blocks;
    bool ok = true;
    for (int t = 0; t < n_tiles && ok; ++t) {
      const int key = (tile_lo + t) * LD_TILE + lane * p.rows_per_box;     // rows past the context: finite values of other tokens
      const int page = min(key / p.block_size, p.max_blocks - 1);
      const int blk = min(max(lane < p.boxes ? __ldg(bt + page) : 0, 0), p.num_blocks - 1);
      const int row = blk * p.block_size + key % p.block_size;
      for (int c = 0; c < p.pieces; ++c) {
        ok = mbar_wait(bar(EMPTY + c), (t & 1) ^ 1u, abort_word, FT_ERR_TIMEOUT_PRODUCER);
        if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
        if (lane == 0) mbar_expect_tx(bar(FULL + c), LD_PIECE);
        __syncwarp();
        if (lane < p.boxes) tma_load_2d(sbase + c * LD_PIECE + lane * p.rows_per_box * 128, &tmC, bar(FULL + c), c * 64, row);
      }
    }
    if (*abort_word) {   // let copies in flight land before the CTA leaves
      const unsigned long long t0 = globaltimer_ns();
      while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc_f16(LD_TILE, N, 1, 0, 0);
      constexpr uint32_t idesc_o = make_idesc_f16(128, N, 1, 1, 0);
      bool ok = true;
      for (int t = 0; t < n_tiles && ok; ++t) {
        for (int c = 0; c < p.pieces; ++c) {
          ok = mbar_wait(bar(FULL + c), t & 1, abort_word, FT_ERR_TIMEOUT_MMA);
          if (!ok) break;
          tc_fence_after();
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            umma_f16_ss(tmem + COL_S, make_smem_desc_sw128(sbase + c * LD_PIECE + kk * 32, 16, 1024),
                        make_smem_desc_sw128(sbase + Cfg::OFF_Q + c * Cfg::Q_PIECE + kk * 32, 16, 1024), idesc_s, (c > 0 || kk > 0) ? 1u : 0u);
          if (c >= p.v_pieces) umma_commit(bar(EMPTY + c));
        }
        if (!ok) break;
        umma_commit(bar(S_FULL));
        ok = mbar_wait(bar(P_FULL), t & 1, abort_word, FT_ERR_TIMEOUT_MMA);
        if (!ok) break;
        tc_fence_after();
        for (int i = 0; i < blocks; ++i) {
#pragma unroll
          for (int kk = 0; kk < LD_TILE / 16; ++kk)
            umma_f16_ss(tmem + COL_O + i * N, make_smem_desc_sw128(sbase + 2 * i * LD_PIECE + kk * 2048, LD_PIECE, 1024),
                        make_smem_desc_sw128(sbase + Cfg::OFF_P + (kk >> 2) * Cfg::Q_PIECE + (kk & 3) * 32, 16, 1024), idesc_o, (t > 0 || kk > 0) ? 1u : 0u);
          umma_commit(bar(EMPTY + 2 * i));
          umma_commit(bar(EMPTY + 2 * i + 1));
        }
        umma_commit(bar(O_DONE));
      }
    }
  } else if (warp >= 4) {
    // ------------------------------------------------------------------ softmax / epilogue
    constexpr int G = LD_GROUP;
    const int ew = warp & 3, r = ew * 32 + lane, group = (warp - 4) >> 2, hg = group * G;    // first head of the group
    float* s_red = reinterpret_cast<float*>(smem + Cfg::OFF_RED) + group * 5 * G;
    float* s_ref = s_red + 4 * G;
    auto group_sync = [&]() { asm volatile("bar.sync %0, 128;" ::"r"(1 + group) : "memory"); };
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(ew * 32) << 16);
    float l_part[G];
#pragma unroll
    for (int g = 0; g < G; ++g) l_part[g] = 0.f;
    if (r < G) s_ref[r] = -INFINITY;
    bool ok = true;
    // every thread runs every iteration down to the named barriers, also after a failed wait
    for (int t = 0; t < n_tiles; ++t) {
      if (ok && !mbar_wait(bar(S_FULL), t & 1, abort_word, FT_ERR_TIMEOUT_EPILOGUE)) ok = false;
      ok = __all_sync(0xffffffffu, ok);
      float s[G];
      {
        uint32_t raw[G];
#pragma unroll
        for (int g = 0; g < G; ++g) raw[g] = 0u;
        if (ok) {
          tc_fence_after();
#pragma unroll
          for (int g = 0; g < G; g += 16) tmem_ld_32x16(lane_addr + COL_S + hg + g, *reinterpret_cast<uint32_t(*)[16]>(&raw[g]));
          tmem_ld_wait();
        }
        const bool valid = (tile_lo + t) * LD_TILE + r < len;
#pragma unroll
        for (int g = 0; g < G; ++g) s[g] = valid ? __uint_as_float(raw[g]) * p.scale_log2 : -INFINITY;
      }
      // maxima over the warp's keys: halve the heads a lane holds while doubling the keys it covers; lane g ends with head g
      {
        float v[G];
#pragma unroll
        for (int g = 0; g < G; ++g) v[g] = s[g];
#pragma unroll
        for (int w = G / 2; w >= 1; w >>= 1) {
          const bool upper = lane & w;
#pragma unroll
          for (int g = 0; g < w; ++g) {
            const float send = upper ? v[g] : v[g + w], keep = upper ? v[g + w] : v[g];
            v[g] = fmaxf(keep, __shfl_xor_sync(0xffffffffu, send, w));
          }
        }
        v[0] = fmaxf(v[0], __shfl_xor_sync(0xffffffffu, v[0], 16));
        if (lane < G) s_red[ew * G + lane] = v[0];
      }
      group_sync();
      // every thread makes the same decision; the references are replaced after all have read them
      const float tile_max = lane < G ? fmaxf(fmaxf(s_red[lane], s_red[G + lane]), fmaxf(s_red[2 * G + lane], s_red[3 * G + lane])) : -INFINITY;
      const float old_ref = lane < G ? s_ref[lane] : 0.f;
      const bool moves = lane < G && tile_max > old_ref + LD_RESCALE;
      const float my_ref = moves ? tile_max : old_ref, my_alpha = moves ? fast_exp2(old_ref - tile_max) : 1.f;   // first tile: 0
      const bool any = __any_sync(0xffffffffu, moves);
      // O of the earlier tiles and the P buffer are free once the products of tile t - 1 have finished
      if (t > 0 && ok && !mbar_wait(bar(O_DONE), (t - 1) & 1, abort_word, FT_ERR_TIMEOUT_EPILOGUE)) ok = false;
      ok = __all_sync(0xffffffffu, ok);
      if (any) {
        float alpha[G];
#pragma unroll
        for (int g = 0; g < G; ++g) {
          alpha[g] = __shfl_sync(0xffffffffu, my_alpha, g);
          l_part[g] *= alpha[g];
        }
        if (t > 0 && ok) {
          tc_fence_after();
          for (int i = 0; i < blocks; ++i)
#pragma unroll
            for (int g0 = 0; g0 < G; g0 += 16) {
              uint32_t ov[16];
              tmem_ld_32x16(lane_addr + COL_O + i * N + hg + g0, ov);
              tmem_ld_wait();
#pragma unroll
              for (int g = 0; g < 16; ++g) ov[g] = __float_as_uint(__uint_as_float(ov[g]) * alpha[g0 + g]);
              tmem_st_32x16(lane_addr + COL_O + i * N + hg + g0, ov);
            }
          tmem_st_wait();
        }
      }
      {
        uint8_t* pb = smem + Cfg::OFF_P + (r >> 6) * Cfg::Q_PIECE;
        const int kc = r & 63;
#pragma unroll
        for (int g = 0; g < G; ++g) {
          const float ref = __shfl_sync(0xffffffffu, my_ref, g);
          const float pv = s[g] == -INFINITY ? 0.f : fast_exp2(s[g] - ref);
          const __nv_bfloat16 pb16 = __float2bfloat16(pv);
          l_part[g] += __bfloat162float(pb16);     // the sum of what the MMA will actually use
          *reinterpret_cast<__nv_bfloat16*>(pb + (hg + g) * 128 + (((kc >> 3) ^ (g & 7)) << 4) + (kc & 7) * 2) = pb16;
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (ok && lane == 0) mbar_arrive(bar(P_FULL));
      group_sync();      // s_red and the old references have been read by all
      if (ew == 0 && lane < G) s_ref[lane] = my_ref;
    }
    if (ok && n_tiles > 0) ok = mbar_wait(bar(O_DONE), (n_tiles - 1) & 1, abort_word, FT_ERR_TIMEOUT_EPILOGUE);
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
#pragma unroll
    for (int g = 0; g < G; ++g) {
      const float ws = warp_sum(l_part[g]);
      if (lane == 0) s_red[ew * G + g] = ws;
    }
    group_sync();
    if (ok)
      for (int i = 0; i < blocks; ++i)
#pragma unroll
        for (int g0 = 0; g0 < G; g0 += 16) {
          uint32_t ov[16];
#pragma unroll
          for (int g = 0; g < 16; ++g) ov[g] = 0u;
          if (n_tiles > 0) {
            tmem_ld_32x16(lane_addr + COL_O + i * N + hg + g0, ov);
            tmem_ld_wait();
          }
          const int d = i * 128 + r;
#pragma unroll
          for (int g = 0; g < 16; ++g) {
            const int h = g0 + g;
            if (hg + h >= heads || d >= p.rank) continue;
            const float l = s_red[h] + s_red[G + h] + s_red[2 * G + h] + s_red[3 * G + h], o = __uint_as_float(ov[g]);
            if (p.n_splits == 1) {
              p.out[b * p.ldo + static_cast<long long>(h0 + hg + h) * p.rank + d] = __float2bfloat16(l > 0.f ? o / l : 0.f);
            } else {
              const long long at = (static_cast<long long>(b) * p.H + h0 + hg + h) * p.n_splits + split;
              p.part_o[at * p.rank + d] = o;
              if (d == 0) { p.part_ml[at * 2] = s_ref[h]; p.part_ml[at * 2 + 1] = l; }
            }
          }
        }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 2) {
    tc_fence_after();
    tmem_dealloc(tmem, Cfg::TMEM_COLS);
  }
  if (threadIdx.x == 0 && *abort_word != 0 && p.status) atomicCAS(p.status, 0, *abort_word);
}

// One block per (head, row): the splits' factors once, then their rows in vectors of four.
constexpr int LC_MAX_SPLITS = 32;
__global__ void __launch_bounds__(128)
latent_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, __nv_bfloat16* __restrict__ out, int H, int rank,
                      long long ldo, int n_splits) {
  __shared__ float s_f[LC_MAX_SPLITS];
  const int h = blockIdx.x, b = blockIdx.y;
  const long long base = (static_cast<long long>(b) * H + h) * n_splits;
  if (threadIdx.x < 32) {
    const int s = threadIdx.x;
    const float m = s < n_splits ? part_ml[(base + s) * 2] : -INFINITY;
    const float mm = warp_max(m);
    const float f = m == -INFINITY ? 0.f : fast_exp2(m - mm);
    const float l = warp_sum(s < n_splits ? part_ml[(base + s) * 2 + 1] * f : 0.f);
    s_f[s] = l > 0.f ? f / l : 0.f;
  }
  __syncthreads();
  for (int d = threadIdx.x * 4; d < rank; d += 512) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < n_splits; ++s) {
      const float f = s_f[s];
      if (f == 0.f) continue;                      // a split without keys left its partial result unwritten or zero
      const float4 o = *reinterpret_cast<const float4*>(part_o + (base + s) * rank + d);
      acc.x += f * o.x; acc.y += f * o.y; acc.z += f * o.z; acc.w += f * o.w;
    }
    *reinterpret_cast<uint2*>(out + b * ldo + static_cast<long long>(h) * rank + d) = make_uint2(pack_bf16x2(acc.x, acc.y), pack_bf16x2(acc.z, acc.w));
  }
}

// out[first + i] = cached row of token i of sequence slot, i < n, for every (slot, first, n) of `spans`; zeros up to the next
// multiple of `pad` rows.
constexpr int LG_BATCH = 4;       // units loaded together
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ cache, const int* __restrict__ block_table, const int* __restrict__ spans,
                     uint4* __restrict__ out, int units, int pad, int block_size, int max_blocks, int num_blocks) {
  const int* span = spans + 3 * blockIdx.y;
  const int n = span[2];
  const int* bt = block_table + static_cast<long long>(span[0]) * max_blocks;
  const long long total = static_cast<long long>((n + pad - 1) / pad * pad) * units;
  uint4* dst = out + static_cast<long long>(span[1]) * units;
  for (long long base = static_cast<long long>(blockIdx.x) * 256 * LG_BATCH; base < total; base += static_cast<long long>(gridDim.x) * 256 * LG_BATCH) {
    uint4 v[LG_BATCH];
#pragma unroll
    for (int j = 0; j < LG_BATCH; ++j) {
      const long long at = base + j * 256 + threadIdx.x;
      const int i = static_cast<int>(at / units), u = static_cast<int>(at - static_cast<long long>(i) * units);
      v[j] = make_uint4(0u, 0u, 0u, 0u);
      if (at < total && i < n) {
        const int page = i / block_size;
        const int blk = min(max(page < max_blocks ? __ldg(bt + page) : 0, 0), num_blocks - 1);
        v[j] = cache[(static_cast<long long>(blk) * block_size + i % block_size) * units + u];
      }
    }
#pragma unroll
    for (int j = 0; j < LG_BATCH; ++j) {
      const long long at = base + j * 256 + threadIdx.x;
      if (at < total) dst[at] = v[j];
    }
  }
}

static bool la_aligned(std::initializer_list<const void*> ps) {
  uintptr_t v = 0;
  for (const void* p : ps) v |= reinterpret_cast<uintptr_t>(p);
  return (v & 15) == 0;
}

}  // namespace ft

using namespace ft;

// The pass between a packed projection and its latent attention (see the top of this file): query heads of q_head elements
// from q_off, their rotated part of rot_pad elements at q_rot; latent and key part of rank_pad + rot_pad from c_off, of
// which rank and 2 * half exist (padding is zero).  packed and cache bf16, or fp32 with f32; all sizes and offsets multiples of
// 8.  Rows n_lat .. keep their rotated query parts in place, the rows ahead of them put theirs into q_lat; the latent and the
// key part go to the page only.
FT_API int ft_latent_finish(void* packed, long long ld, void* q_lat, int n_lat, const int* pos, const int* slots, const int* block_table,
                            void* cache, const float* weight, const void* table, int rows, int H, int q_off, int q_head, int q_rot,
                            int c_off, int rank_pad, int rank, int rot_pad, int half, int positions, float eps, int f32, int block_size,
                            int max_blocks, int num_blocks, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(packed && pos && slots && block_table && cache && weight && table && (q_lat || n_lat == 0), "ft_latent_finish: null pointer");
  FT_REQUIRE(((q_off | q_head | q_rot | c_off | rank_pad | rot_pad) & 7) == 0 && ld % 8 == 0, "ft_latent_finish: sizes must be multiples of 8");
  FT_REQUIRE(H > 0 && q_off >= 0 && c_off >= 0 && q_rot >= 0 && q_rot + rot_pad <= q_head && rank > 0 && rank <= rank_pad && half > 0 &&
                 2 * half <= rot_pad && positions > 0 && n_lat >= 0 && n_lat <= rows,
             "ft_latent_finish: bad shape");
  FT_REQUIRE(q_off + static_cast<long long>(H) * q_head <= ld && c_off + rank_pad + rot_pad <= ld, "ft_latent_finish: the row is too short");
  FT_REQUIRE(la_aligned({packed, q_lat, cache, weight}) && (reinterpret_cast<uintptr_t>(table) & 7) == 0 && block_size > 0 && max_blocks > 0 && num_blocks > 0,
             "ft_latent_finish: pointers must be 16-byte aligned");
  if (rows <= 0) return FT_E_OK;
  LatentFinishParams p;
  p.packed = packed; p.q_lat = q_lat; p.pos = pos; p.slots = slots; p.block_table = block_table; p.cache = cache; p.weight = weight;
  p.table = static_cast<const float2*>(table); p.ld = ld; p.rows = rows; p.n_lat = n_lat; p.H = H; p.q_off = q_off; p.q_head = q_head;
  p.q_rot = q_rot; p.c_off = c_off; p.rank_pad = rank_pad; p.rank = rank; p.rot_pad = rot_pad; p.half = half; p.positions = positions;
  p.eps = eps; p.block_size = block_size; p.max_blocks = max_blocks; p.num_blocks = num_blocks;
  const int grid = (rows + LF_ROWS - 1) / LF_ROWS;
  int threads = 32 * LF_ROWS + (H * (rot_pad / 8) + 31) / 32 * 32;
  if (threads > LF_MAX_THREADS) threads = LF_MAX_THREADS;
  if (f32) latent_finish_kernel<float><<<grid, threads, 0, stream>>>(p);
  else latent_finish_kernel<__nv_bfloat16><<<grid, threads, 0, stream>>>(p);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// Decode attention over latent rows (see the top of this file): q [B, H, width] bf16, cache [num_blocks, block_size, width], out
// [B, H, rank] (row stride ldo), width and rank multiples of 16, width up to 576 and rank up to 512.  Row b reads its first
// ctx_len[b] tokens of sequence row_slot[b] (null: b).  scratch: B * H * n_splits * (rank + 2) floats when n_splits > 1.  Page
// sizes: a divisor of 128 of at least 8, or a multiple of 128.
FT_API int ft_latent_decode(const void* q, const void* cache, const int* block_table, const int* row_slot, const int* ctx_len, void* out,
                            float* scratch, int B, int H, int width, int rank, long long ldo, int block_size, int max_blocks,
                            int num_blocks, float scale, int n_splits, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(q && cache && block_table && ctx_len && out, "ft_latent_decode: null pointer");
  FT_REQUIRE(H > 0 && width >= 16 && width % 16 == 0 && width <= LD_MAX_PIECES * 64 && rank >= 16 && rank % 16 == 0 && rank <= width && rank <= 512,
             "ft_latent_decode: rows of %d with a latent of %d", width, rank);
  FT_REQUIRE(block_size >= 8 && (LD_TILE % block_size == 0 || block_size % LD_TILE == 0) && max_blocks > 0 && num_blocks > 0 &&
                 static_cast<long long>(num_blocks) * block_size < (1ll << 31), "ft_latent_decode: page size %d", block_size);
  FT_REQUIRE(n_splits >= 1 && n_splits <= LC_MAX_SPLITS && (n_splits == 1 || scratch), "ft_latent_decode: %d splits", n_splits);
  FT_REQUIRE(la_aligned({q, cache, out, scratch}) && ldo % 8 == 0 && ldo >= static_cast<long long>(H) * rank, "ft_latent_decode: pointers must be 16-byte aligned");
  if (B <= 0) return FT_E_OK;
  FT_REQUIRE(B < 65536, "ft_latent_decode: %d rows", B);
  LatentDecodeParams p;
  p.q = static_cast<const __nv_bfloat16*>(q); p.block_table = block_table; p.row_slot = row_slot; p.ctx_len = ctx_len;
  p.out = static_cast<__nv_bfloat16*>(out); p.part_o = scratch;
  p.part_ml = scratch ? scratch + static_cast<long long>(B) * H * n_splits * rank : nullptr;
  p.ldo = ldo; p.H = H; p.width = width; p.rank = rank; p.v_pieces = 2 * ((rank + 127) / 128);
  p.pieces = (width + 63) / 64;
  if (p.pieces < p.v_pieces) p.pieces = p.v_pieces;          // a piece past the row: zeros
  p.block_size = block_size; p.rows_per_box = block_size < LD_TILE ? block_size : LD_TILE; p.boxes = LD_TILE / p.rows_per_box;
  p.max_blocks = max_blocks; p.num_blocks = num_blocks; p.n_splits = n_splits;
  p.scale_log2 = scale * 1.4426950408889634f; p.status = device_status_word(device);
  CUtensorMap tc;
  if (int rc = make_tmap_2d(&tc, cache, 2, width, static_cast<uint64_t>(num_blocks) * block_size, static_cast<uint64_t>(width) * 2, 64, p.rows_per_box, 3))
    return rc;
  const int N = H <= 16 ? 16 : 32;
  const dim3 grid(n_splits, (H + N - 1) / N, B);
#define FT_LD(NN)                                                                                                                   \
  {                                                                                                                                 \
    static bool attr_set[64] = {false};                                                                                             \
    if (!attr_set[device]) {                                                                                                        \
      FT_CUDA_CHECK(cudaFuncSetAttribute(latent_decode_kernel<NN>, cudaFuncAttributeMaxDynamicSharedMemorySize, LdCfg<NN>::SMEM_BYTES)); \
      attr_set[device] = true;                                                                                                      \
    }                                                                                                                               \
    latent_decode_kernel<NN><<<grid, LdCfg<NN>::THREADS, LdCfg<NN>::SMEM_BYTES, stream>>>(tc, p);                                           \
  }
  if (N == 16) FT_LD(16) else FT_LD(32)
#undef FT_LD
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  if (n_splits > 1) {
    latent_combine_kernel<<<dim3(H, B), 128, 0, stream>>>(p.part_o, p.part_ml, p.out, H, rank, ldo, n_splits);
    FT_CUDA_CHECK(cudaGetLastError());
    count_launch();
  }
  return FT_E_OK;
}

// The cached rows of contexts, contiguous: spans int32 [n_spans, 3] (sequence slot, first row of out, tokens), rows of
// row_bytes (a multiple of 16); every span is filled up with zero rows to a multiple of `pad`.  longest: most tokens of a span.
FT_API int ft_latent_gather(const void* cache, const int* block_table, const int* spans, int n_spans, int longest, void* out, int row_bytes,
                            int pad, int block_size, int max_blocks, int num_blocks, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(cache && block_table && spans && out && row_bytes > 0 && row_bytes % 16 == 0 && pad > 0 && la_aligned({cache, out}), "ft_latent_gather: null or unaligned pointer");
  FT_REQUIRE(block_size > 0 && max_blocks > 0 && num_blocks > 0 && n_spans < 65536, "ft_latent_gather: bad shape");
  if (n_spans <= 0 || longest <= 0) return FT_E_OK;
  const long long most = static_cast<long long>((longest + pad - 1) / pad * pad) * (row_bytes / 16);
  long long gx = (most + 256 * LG_BATCH - 1) / (256 * LG_BATCH);
  const long long cap = sm_count(device) * 32ll / n_spans + 1;
  if (gx > cap) gx = cap;
  latent_gather_kernel<<<dim3(static_cast<unsigned>(gx), n_spans), 256, 0, stream>>>(static_cast<const uint4*>(cache), block_table, spans,
                                                                                     static_cast<uint4*>(out), row_bytes / 16, pad, block_size, max_blocks, num_blocks);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}
