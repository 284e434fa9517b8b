// Paged KV cache on the device: block tables, append, and single-token decode attention.
//
// The reference keeps its paged cache as a host-side data structure that no kernel consumes
// (PagePool / PagedKVCache / PagedAttentionManager, ferrotorch-nn/src/paged_attention.rs:73-532)
// and its GPU decode path re-runs the whole prefix (ferrotorch-llama/src/gpu.rs:549-788).  Here
// the cache is two device arrays [num_blocks, block_size, n_kv_heads, head_dim] (bf16) and an
// int32 block table [batch, max_blocks_per_seq]; token t of sequence b lives in block
// table[b][t / block_size] at row t % block_size.
//
//   ft_kv_append        scatter new K/V rows (a prefill chunk or one decode token per sequence)
//                       into the cache through the block table.
//   ft_paged_decode     one query token per row: softmax(scale * q K^T) V over the cached
//                       context, GQA (all query heads of a KV group share one pass over K/V),
//                       flash-decoding split over the context with a second combine pass, and an
//                       optional output gate per head.
//                       A row may see a window of the most recent keys only, or those of its own chunk; a
//                       bias that grows with the distance may be taken off the scores, and a learned number
//                       per head (a sink) may join the denominator.  Ahead of a window it may see the means of
//                       whole blocks of keys and values.
//   ft_pool_blocks      these means, of the blocks that end among the rows of a step.
//   ft_paged_rows       the same for any mixture of rows (each with its own sequence and number of
//                       visible keys), any head sizes, bf16 or fp32: the exact, simple kernel.
// Decode attention is bandwidth bound (every cached byte is read once per step).  Key / value head
// sizes up to 128 (multiples of 16; they may differ) run on the tensor-core kernel
// (paged_decode_tc_kernel: cp.async rows -> shared memory -> tcgen05.mma).  The CUDA-core kernel for
// equal sizes of 64 or 128 reads K with one key per lane (full rows, no shuffles in the dot products)
// and V with one row per warp step; it serves size 64, and queries that are not 16-byte aligned.
#include "attn_row.cuh"
#include "ft_host.h"
#include "row_vec.cuh"

namespace ft {

constexpr int PD_THREADS = 128;
constexpr int PD_WARPS = PD_THREADS / 32;

// k_new / v_new: rows of kv16 / vv16 16-byte units (all KV heads of a token) with token strides ldk16 / ldv16 units.
// Token i goes to sequence seq_ids[i] (or i / tokens_per_seq when null) at position pos[i].
__global__ void kv_append_kernel(const uint4* __restrict__ k_new, const uint4* __restrict__ v_new, uint4* __restrict__ k_cache,
                                 uint4* __restrict__ v_cache, const int* __restrict__ block_table,
                                 const int* __restrict__ pos, const int* __restrict__ seq_ids, int T, int tokens_per_seq,
                                 int kv16, int vv16, long long ldk16, long long ldv16, int block_size, int max_blocks,
                                 int num_blocks) {
  for (int t = blockIdx.x; t < T; t += gridDim.x) {
    const int b = seq_ids ? seq_ids[t] : t / tokens_per_seq;
    const int p = pos[t];
    const int blk = block_table[static_cast<long long>(b) * max_blocks + p / block_size];
    if (blk < 0 || blk >= num_blocks) continue;  // host validates; never write out of range
    const long long token = static_cast<long long>(blk) * block_size + p % block_size;
    for (int i = threadIdx.x; i < max(kv16, vv16); i += blockDim.x) {
      if (i < kv16) k_cache[token * kv16 + i] = k_new[t * ldk16 + i];
      if (i < vv16) v_cache[token * vv16 + i] = v_new[t * ldv16 + i];
    }
  }
}

// Row i ends a block when (pos[i] + 1) % pool == 0: the means of its pool keys and values (their rows are in the cache) go to the
// block's place.  A thread owns eight elements of a token's keys or values; a CTA takes `walk` (up to 32) consecutive rows, of
// which a portion has few that end a block.
constexpr int PB_THREADS = 128;
constexpr int PB_BATCH = 8;       // rows loaded together
template <typename T>
__global__ void __launch_bounds__(PB_THREADS)
pool_blocks_kernel(const T* __restrict__ k_cache, const T* __restrict__ v_cache, T* __restrict__ k_pool, T* __restrict__ v_pool,
                   const int* __restrict__ block_table, const int* __restrict__ pos, const int* __restrict__ slots, int rows, int walk, int kw, int vw,
                   int pool, int per_page, int block_size, int max_blocks, int num_blocks) {
  const float inv = 1.f / static_cast<float>(pool);
  const int lane = threadIdx.x & 31, mine = blockIdx.x * walk + lane;
  const bool there = lane < walk && mine < rows;
  const int my_pos = there ? pos[mine] : 0, my_slot = there ? slots[mine] : 0;
  for (unsigned ends = __ballot_sync(0xffffffffu, there && (my_pos + 1) % pool == 0); ends; ends &= ends - 1) {
    const int at = __ffs(ends) - 1, last = __shfl_sync(0xffffffffu, my_pos, at);
    const int* bt = block_table + static_cast<long long>(__shfl_sync(0xffffffffu, my_slot, at)) * max_blocks;
    const int page = last / block_size, first = last + 1 - pool;
    if (page >= max_blocks || bt[page] < 0 || bt[page] >= num_blocks) continue;   // a row of no sequence
    const long long dst = static_cast<long long>(bt[page]) * per_page + (last / pool - page * block_size / pool);
    for (int i = (blockIdx.y * PB_THREADS + threadIdx.x) * 8; i < kw + vw; i += gridDim.y * PB_THREADS * 8) {
      const bool is_k = i < kw;
      const int c = is_k ? i : i - kw, width = is_k ? kw : vw;
      const T* src = is_k ? k_cache : v_cache;
      float sum[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) sum[e] = 0.f;
      for (int j0 = 0; j0 < pool; j0 += PB_BATCH) {
        uint4 raw[PB_BATCH][sizeof(T) / 2];
#pragma unroll
        for (int j = 0; j < PB_BATCH; ++j) {            // past the end: the last row again
          const int p = first + min(j0 + j, pool - 1);
          const int blk = min(max(__ldg(bt + p / block_size), 0), num_blocks - 1);
          raw_load(src + (static_cast<long long>(blk) * block_size + p % block_size) * width + c, raw[j]);
        }
#pragma unroll
        for (int j = 0; j < PB_BATCH; ++j) {
          if (j0 + j >= pool) continue;
          float f[8];
          raw_unpack(raw[j], f);
#pragma unroll
          for (int e = 0; e < 8; ++e) sum[e] += f[e];
        }
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) sum[e] *= inv;
      store8((is_k ? k_pool : v_pool) + dst * width + c, sum);
    }
  }
}

// grid (n_splits, Hkv, B).  Each CTA covers tiles of 32 keys, strided over its warps, inside its
// slice of the context; partial (m, l, o) per (b, q head, split) go to scratch when n_splits > 1.
// Scores: lane j owns key j of the tile and reads its whole row (all loads issued before the
// math).  PV: the two half-warps take even / odd keys, each lane owns 8 (D=128) or 4 (D=64)
// output dims, V rows are read 8 keys at a time with 16-byte (8-byte) loads.
template <int D, int G>
__global__ void __launch_bounds__(PD_THREADS)
paged_decode_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k_cache,
                    const __nv_bfloat16* __restrict__ v_cache, const int* __restrict__ block_table,
                    const int* __restrict__ row_slot, const int* __restrict__ ctx_len, __nv_bfloat16* __restrict__ out,
                    float* __restrict__ part_o, float* __restrict__ part_ml, int Hq, int Hkv, long long ldq, long long ldo,
                    int block_size, int max_blocks, int num_blocks, float scale_log2, int n_splits, KeyRange range,
                    const float* __restrict__ slopes, const float* __restrict__ sink, HeadGate gate, float out_scale) {
  constexpr int DV = D / 16;  // dims per lane in the PV phase (half-warp covers D)
  const int split = blockIdx.x, kvh = blockIdx.y, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int half = lane >> 4, hl = lane & 15;
  const int len = ctx_len[b];
  const int first = range.first_visible(len);
  const int tiles_end = (len + 31) >> 5;
  const int tiles_per_split = (tiles_end - (first >> 5) + n_splits - 1) / n_splits;
  const int tile_lo = (first >> 5) + split * tiles_per_split, tile_hi = min(tiles_end, tile_lo + tiles_per_split);

  __shared__ __align__(16) float s_q[G][D];          // q * scale * log2(e)
  __shared__ float s_p[PD_WARPS][G][32];             // probabilities of the current tile
  __shared__ float s_m[PD_WARPS][G], s_l[PD_WARPS][G];
  __shared__ __align__(16) float s_o[PD_WARPS][G][D];

  for (int i = threadIdx.x; i < G * D; i += blockDim.x) {
    const int g = i / D, d = i - g * D;
    s_q[g][d] = __bfloat162float(q[static_cast<long long>(b) * ldq + static_cast<long long>(kvh * G + g) * D + d]) * scale_log2;
  }
  __syncthreads();

  float m[G], l[G], o[G][DV], slope[G];
#pragma unroll
  for (int g = 0; g < G; ++g) {
    m[g] = -INFINITY; l[g] = 0.f;
    slope[g] = slopes ? slopes[kvh * G + g] * ATT_LOG2E : 0.f;
#pragma unroll
    for (int j = 0; j < DV; ++j) o[g][j] = 0.f;
  }
  const int* bt = block_table + static_cast<long long>(row_slot ? row_slot[b] : b) * max_blocks;
  const long long row_stride = static_cast<long long>(Hkv) * D;
  const long long head_off = static_cast<long long>(kvh) * D;

  for (int tile = tile_lo + warp; tile < tile_hi; tile += PD_WARPS) {
    const int key0 = tile << 5;
    // ---- scores: lane j owns key key0 + j; issue the whole row's loads, then the dot products
    const int key = key0 + lane;
    const bool valid = key < len && key >= first;
    float s[G];
#pragma unroll
    for (int g = 0; g < G; ++g) s[g] = 0.f;
    {
      const int kk = key < len ? key : key0;
      int blk = bt[kk / block_size];
      blk = min(max(blk, 0), num_blocks - 1);
      const uint4* kr = reinterpret_cast<const uint4*>(
          k_cache + (static_cast<long long>(blk) * block_size + kk % block_size) * row_stride + head_off);
      uint4 kv[D / 8];
#pragma unroll
      for (int c = 0; c < D / 8; ++c) kv[c] = __ldg(kr + c);
#pragma unroll
      for (int c = 0; c < D / 8; ++c) {
        const float2 k0 = unpack_bf16x2(kv[c].x), k1 = unpack_bf16x2(kv[c].y), k2 = unpack_bf16x2(kv[c].z),
                     k3 = unpack_bf16x2(kv[c].w);
#pragma unroll
        for (int g = 0; g < G; ++g) {
          const float4 qa = *reinterpret_cast<const float4*>(&s_q[g][c * 8]);
          const float4 qb = *reinterpret_cast<const float4*>(&s_q[g][c * 8 + 4]);
          s[g] += k0.x * qa.x + k0.y * qa.y + k1.x * qa.z + k1.y * qa.w + k2.x * qb.x + k2.y * qb.y + k3.x * qb.z + k3.y * qb.w;
        }
      }
    }
    // ---- online softmax per head across the 32 lanes
    float alpha[G];
#pragma unroll
    for (int g = 0; g < G; ++g) {
      const float sv = valid ? s[g] - slope[g] * static_cast<float>(len - 1 - key) : -INFINITY;
      const float mx = warp_max(sv);
      const float m_new = fmaxf(m[g], mx);
      const float pv = valid ? fast_exp2(sv - m_new) : 0.f;
      alpha[g] = fast_exp2(m[g] - m_new);  // exp2(-inf) = 0 on the first tile
      l[g] = l[g] * alpha[g] + warp_sum(pv);
      m[g] = m_new;
      s_p[warp][g][lane] = pv;
#pragma unroll
      for (int j = 0; j < DV; ++j) o[g][j] *= alpha[g];
    }
    __syncwarp();
    // ---- O += P V: half-warp `half` takes keys key0 + 2*i + half; 8 keys (per half) in flight
    const int n_keys = min(32, len - key0);
    for (int i0 = 0; i0 < 16; i0 += 8) {
      if (2 * i0 >= n_keys) break;
      uint4 vv[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int j = 2 * (i0 + i) + half;
        const int kj = key0 + min(j, n_keys - 1);
        int blk = bt[kj / block_size];
        blk = min(max(blk, 0), num_blocks - 1);
        const __nv_bfloat16* vr = v_cache + (static_cast<long long>(blk) * block_size + kj % block_size) * row_stride +
                                  head_off + hl * DV;
        if constexpr (DV == 8) {
          vv[i] = __ldg(reinterpret_cast<const uint4*>(vr));
        } else {
          const uint2 t = __ldg(reinterpret_cast<const uint2*>(vr));
          vv[i] = make_uint4(t.x, t.y, 0u, 0u);
        }
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int j = 2 * (i0 + i) + half;
        if (j < n_keys) {
          float f[8];
          const float2 a0 = unpack_bf16x2(vv[i].x), a1 = unpack_bf16x2(vv[i].y);
          f[0] = a0.x; f[1] = a0.y; f[2] = a1.x; f[3] = a1.y;
          if constexpr (DV == 8) {
            const float2 a2 = unpack_bf16x2(vv[i].z), a3 = unpack_bf16x2(vv[i].w);
            f[4] = a2.x; f[5] = a2.y; f[6] = a3.x; f[7] = a3.y;
          }
#pragma unroll
          for (int g = 0; g < G; ++g) {
            const float pj = s_p[warp][g][j];
#pragma unroll
            for (int e = 0; e < DV; ++e) o[g][e] += pj * f[e];
          }
        }
      }
    }
    __syncwarp();
  }

  // ---- combine the two half-warps, then the warps of this CTA
#pragma unroll
  for (int g = 0; g < G; ++g) {
#pragma unroll
    for (int e = 0; e < DV; ++e) o[g][e] += __shfl_xor_sync(0xffffffffu, o[g][e], 16);
    if (lane == 0) { s_m[warp][g] = m[g]; s_l[warp][g] = l[g]; }
    if (half == 0) {
#pragma unroll
      for (int e = 0; e < DV; ++e) s_o[warp][g][hl * DV + e] = o[g][e];
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < G * D; i += blockDim.x) {
    const int g = i / D, d = i - g * D;
    float mm = -INFINITY;
#pragma unroll
    for (int w = 0; w < PD_WARPS; ++w) mm = fmaxf(mm, s_m[w][g]);
    float ll = 0.f, acc = 0.f;
#pragma unroll
    for (int w = 0; w < PD_WARPS; ++w) {
      const float sc = (s_m[w][g] == -INFINITY) ? 0.f : fast_exp2(s_m[w][g] - mm);
      ll += s_l[w][g] * sc;
      acc += s_o[w][g][d] * sc;
    }
    const int hq = kvh * G + g;
    if (n_splits == 1) {
      sink_join(sink, hq, mm, ll, acc);
      out[static_cast<long long>(b) * ldo + static_cast<long long>(hq) * D + d] =
          __float2bfloat16(ll > 0.f ? acc / ll * out_scale * head_gate_bf16(gate, b, hq, d) : 0.f);
    } else {
      const long long pidx = (static_cast<long long>(b) * Hq + hq) * n_splits + split;
      part_o[pidx * D + d] = acc;
      if (d == 0) { part_ml[pidx * 2] = mm; part_ml[pidx * 2 + 1] = ll; }
    }
  }
}

__global__ void paged_decode_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                            __nv_bfloat16* __restrict__ out, int Hq, int D, long long ldo, int n_splits,
                                            const float* __restrict__ sink, HeadGate gate, float out_scale) {
  const int hq = blockIdx.x, b = blockIdx.y;
  const long long base = (static_cast<long long>(b) * Hq + hq) * n_splits;
  float mm = -INFINITY;
  for (int s = 0; s < n_splits; ++s) mm = fmaxf(mm, part_ml[(base + s) * 2]);
  for (int d = threadIdx.x; d < D; d += blockDim.x) {
    float ll = 0.f, acc = 0.f;
    for (int s = 0; s < n_splits; ++s) {
      const float ms = part_ml[(base + s) * 2];
      const float sc = (ms == -INFINITY) ? 0.f : fast_exp2(ms - mm);
      ll += part_ml[(base + s) * 2 + 1] * sc;
      acc += part_o[(base + s) * D + d] * sc;
    }
    float m = mm;
    sink_join(sink, hq, m, ll, acc);
    out[static_cast<long long>(b) * ldo + static_cast<long long>(hq) * D + d] =
        __float2bfloat16(ll > 0.f ? acc / ll * out_scale * head_gate_bf16(gate, b, hq, d) : 0.f);
  }
}


// ----------------------------------------------------------------------------- tensor-core decode
// The decode kernel for key and value head sizes up to 128 (any page size).  Head sizes below the tile's
// (64 or 128 for keys, 128 for values: an MMA with 64 rows lays its accumulator out differently) leave
// zeroed columns in the operand tiles.  A CTA owns one (sequence, KV head, context
// split) and walks its keys in tiles of 128; all query heads of the KV group ride along as the
// (padded) 16-wide N dimension of two small MMAs per tile:
//     S^T[key, head] = K_tile[key, :] . Q[head, :]          (M = 128 keys, N = 16, K = head_dim)
//     O^T[dim, head] += V_tile^T[dim, key] . P^T[key, head]  (M = head_dim rows, N = 16, K = 128 keys)
// so the cached K and V rows go from HBM to shared memory with 16-byte cp.async copies (a page of
// 16 tokens x one head is only 2 KB per 64-wide half, too small a box for TMA to move at
// bandwidth; four loader warps keep three 64 KB tiles in flight instead) and from there straight
// into the tensor core: no per-element CUDA-core arithmetic on the cache at all.  The four softmax warps (thread r = key r of the tile) only handle the
// 128 x G scores: tile maximum over the keys (warp shuffles + one exchange through shared
// memory), lazy rescale of O^T in tensor memory, P^T as bf16 into a small shared-memory operand.
//   warp 1: MMA issuer     warp 2: TMEM allocator     warps 4-7: softmax / epilogue
//   warps 8-11: loaders (block-table lookups, cp.async into the 128-byte-swizzled operand
//   layout, rows past the context zero-filled; 3-stage ring of {K, V} tiles)
// Partial results use the same (m, l, o) scratch layout as paged_decode_kernel, so the combine
// pass is shared.  All waits are bounded.
constexpr int PT_THREADS = 384;
constexpr int PT_LOADERS = 128;  // warps 8-11
constexpr int PT_TILE = 128;   // keys per tile
constexpr int PT_STAGES = 3;
constexpr int PT_N = 16;       // MMA N: query heads of the group, zero-padded
constexpr float PT_RESCALE = 8.f;

constexpr int PT_VD = 128;     // rows of O^T

template <int HD>
struct PtCfg {  // HD: width of the K tile (64 or 128)
  static constexpr int K_BYTES = PT_TILE * HD * 2;
  static constexpr int V_BYTES = PT_TILE * PT_VD * 2;
  static constexpr int STAGE_BYTES = K_BYTES + V_BYTES;
  static constexpr int CHUNK = PT_TILE * 128;             // one 64-wide column chunk of a tile
  static constexpr int Q_BYTES = PT_N * HD * 2;           // Q^T operand: 16 rows x key head size
  static constexpr int P_BYTES = PT_N * PT_TILE * 2;      // P^T operand: 16 rows x 128 keys
  static constexpr int OFF_Q = PT_STAGES * STAGE_BYTES;
  static constexpr int OFF_P = OFF_Q + Q_BYTES;           // two buffers
  static constexpr int OFF_RED = OFF_P + 2 * P_BYTES;     // [4 warps][16] floats
  static constexpr int OFF_BAR = OFF_RED + 4 * PT_N * 4;
  static constexpr int SMEM_BYTES = OFF_BAR + 256 + 1024;
};

// G: query heads of a group, rounded up to 1 / 2 / 4 / 8 / 16 (g_real of them exist).  D, Dv: key and value
// head sizes, multiples of 16.
template <int HD, int G>
__global__ void __launch_bounds__(PT_THREADS, 1)
paged_decode_tc_kernel(const __nv_bfloat16* __restrict__ k_cache, const __nv_bfloat16* __restrict__ v_cache,
                       const __nv_bfloat16* __restrict__ q, const int* __restrict__ block_table,
                       const int* __restrict__ row_slot, const int* __restrict__ ctx_len, __nv_bfloat16* __restrict__ out,
                       float* __restrict__ part_o, float* __restrict__ part_ml, int Hq, int Hkv, int D, int Dv, int g_real,
                       long long ldq, long long ldo, int block_size, int max_blocks, int num_blocks, float scale_log2,
                       int n_splits, KeyRange range, PooledKeys pooled, const float* __restrict__ slopes, const float* __restrict__ sink,
                       HeadGate gate, float out_scale, int* status) {
  using Cfg = PtCfg<HD>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  const uint32_t sbase = smem_u32(smem);
  const uint32_t sQ = sbase + Cfg::OFF_Q, sP = sbase + Cfg::OFF_P;
  float* s_red = reinterpret_cast<float*>(smem + Cfg::OFF_RED);
  enum { KV_FULL = 0, ST_EMPTY = KV_FULL + PT_STAGES, S_FULL = ST_EMPTY + PT_STAGES,
         P_FULL = S_FULL + 2, O_DONE = P_FULL + 2, NBARS = O_DONE + 1 };
  const uint32_t bar0 = sbase + Cfg::OFF_BAR;
  auto bar = [&](int i) { return bar0 + 8u * i; };
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + Cfg::OFF_BAR + 8 * NBARS);
  volatile int* abort_word = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int split = blockIdx.x, kvh = blockIdx.y, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int len = ctx_len[b];
  const int first = range.first_visible(len);
  // tiles of pooled blocks, then tiles of keys from the first visible one's on; tile_lo counts in this order
  const int n_pool = pooled.count(first), pool_tiles = (n_pool + PT_TILE - 1) / PT_TILE;
  const int key_tile = first / PT_TILE - pool_tiles;             // tile t holds keys from (key_tile + t) * PT_TILE on
  const int tiles_all = pool_tiles + max(0, (len + PT_TILE - 1) / PT_TILE - first / PT_TILE);
  const int tiles_per_split = (tiles_all + n_splits - 1) / n_splits;
  const int tile_lo = split * tiles_per_split;
  const int n_tiles = max(0, min(tiles_all, tile_lo + tiles_per_split) - tile_lo);

  if (threadIdx.x == 0) {
    *abort_word = 0;
    for (int s = 0; s < PT_STAGES; ++s) {
      mbar_init(bar(KV_FULL + s), PT_LOADERS);   // every loader thread arrives once its copies have landed
      mbar_init(bar(ST_EMPTY + s), 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(bar(S_FULL + s), 1);
      mbar_init(bar(P_FULL + s), 4);
    }
    mbar_init(bar(O_DONE), 1);
    fence_mbar_init();
  }
  if (warp == 2) {
    tmem_alloc(smem_u32(tmem_slot), 64);
    tmem_relinquish();
  }
  // Q^T operand (bf16, rows past the group zero; the scale is applied to the fp32 scores) and zeroed
  // P^T buffers, written by all threads.  Head sizes below the tile's: the columns that the loaders
  // never write are zeroed in every stage.
  for (int i = threadIdx.x; i < (Cfg::Q_BYTES + 2 * Cfg::P_BYTES) / 16; i += blockDim.x)
    reinterpret_cast<uint4*>(smem + Cfg::OFF_Q)[i] = make_uint4(0u, 0u, 0u, 0u);
  if (D < HD || Dv < PT_VD)
    for (int i = threadIdx.x; i < PT_STAGES * Cfg::STAGE_BYTES / 16; i += blockDim.x)
      reinterpret_cast<uint4*>(smem)[i] = make_uint4(0u, 0u, 0u, 0u);
  __syncthreads();
  for (int i = threadIdx.x; i < g_real * (D / 8); i += blockDim.x) {
    const int g = i / (D / 8), j = i - g * (D / 8);  // 16-byte chunk j of head g
    const uint4 raw = *reinterpret_cast<const uint4*>(q + static_cast<long long>(b) * ldq +
                                                      static_cast<long long>(kvh * g_real + g) * D + j * 8);
    const int c = j >> 3, jj = j & 7;                // 64-wide chunk, 16-byte unit inside it
    *reinterpret_cast<uint4*>(smem + Cfg::OFF_Q + c * (PT_N * 128) + g * 128 + ((jj ^ (g & 7)) << 4)) = raw;
  }
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t COL_S = 0, COL_O = 32;

  if (warp >= 8) {
    // ------------------------------------------------------------------ loaders
    // Thread lt copies 16-byte unit (lt & 15) of rows (lt >> 4) + 8 i, i = 0..15, of the K tile
    // and of the V tile: 16 consecutive threads read one 256-byte cache row.
    const int lt = threadIdx.x - 256;
    const int unit = lt & 15, row0 = lt >> 4;
    const int* bt = block_table + static_cast<long long>(row_slot ? row_slot[b] : b) * max_blocks;
    const bool has_k = unit * 8 < D, has_v = unit * 8 < Dv;   // this thread's 16-byte column exists
    const uint32_t chunk_off = static_cast<uint32_t>(unit >> 3) * Cfg::CHUNK;
    constexpr int AHEAD = PT_STAGES - 1;
    bool ok = true;
    for (int t = 0; t < n_tiles + AHEAD; ++t) {
      // First hand over tile t - AHEAD (groups are committed once per iteration, so "at most
      // AHEAD - 1 groups pending" means its copies have landed).  This must come before the
      // wait below: the MMA warp needs tile t - AHEAD + 1 ... to make progress towards freeing
      // the stage this iteration is about to wait for.
      if (t >= AHEAD) {
        asm volatile("cp.async.wait_group %0;" ::"n"(AHEAD - 1) : "memory");
        fence_proxy_async_smem();
        if (ok) mbar_arrive(bar(KV_FULL + (t - AHEAD) % PT_STAGES));
      }
      if (t < n_tiles && ok) {
        const int st = t % PT_STAGES;
        ok = mbar_wait(bar(ST_EMPTY + st), ((t / PT_STAGES) & 1) ^ 1u, abort_word, FT_ERR_TIMEOUT_PRODUCER);
        if (ok) {
          const uint32_t sK = sbase + st * Cfg::STAGE_BYTES + chunk_off, sV = sK + Cfg::K_BYTES;
          auto copy = [&](int row, const __nv_bfloat16* k, const __nv_bfloat16* v, long long src, bool there) {
            const uint32_t dst = static_cast<uint32_t>(row) * 128u + (static_cast<uint32_t>((unit & 7) ^ (row & 7)) << 4);
            const uint32_t nbytes = there ? 16u : 0u;       // rows past the context are zero-filled
            if (has_k)
              asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(sK + dst),
                           "l"(k + src * D + unit * 8), "r"(nbytes) : "memory");
            if (has_v)
              asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(sV + dst),
                           "l"(v + src * Dv + unit * 8), "r"(nbytes) : "memory");
          };
          if (tile_lo + t < pool_tiles) {
            const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(pooled.k);
            const __nv_bfloat16* vp = static_cast<const __nv_bfloat16*>(pooled.v);
#pragma unroll 4
            for (int i = 0; i < 16; ++i) {
              const int row = row0 + 8 * i, block = (tile_lo + t) * PT_TILE + row;
              const bool there = block < n_pool;
              const long long src = there ? pooled.row(block, bt, block_size, max_blocks, num_blocks) * Hkv + kvh : 0;
              copy(row, kp, vp, src, there);
            }
          } else {
            const int key0 = (key_tile + tile_lo + t) * PT_TILE;
#pragma unroll
            for (int i = 0; i < 16; ++i) {
              const int row = row0 + 8 * i;
              const int key = key0 + row;
              const int page = key / block_size;
              int blk = (key < len && page < max_blocks) ? __ldg(bt + page) : 0;
              blk = min(max(blk, 0), num_blocks - 1);
              copy(row, k_cache, v_cache, (static_cast<long long>(blk) * block_size + key % block_size) * Hkv + kvh, key < len);
            }
          }
        }
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0 && n_tiles > 0) {
      constexpr uint32_t idesc_qk = make_idesc_f16(PT_TILE, PT_N, 1, 0, 0);   // keys x heads, both K-major
      constexpr uint32_t idesc_pv = make_idesc_f16(PT_VD, PT_N, 1, 1, 0);     // dims x heads, A (V^T) MN-major
      auto issue_qk = [&](int t) {
        const uint32_t sK = sbase + (t % PT_STAGES) * Cfg::STAGE_BYTES;
        const uint32_t d = tmem_base + COL_S + (t & 1) * PT_N;
#pragma unroll
        for (int kk = 0; kk < HD / 16; ++kk) {
          const uint32_t ko = (kk >> 2) * Cfg::CHUNK + (kk & 3) * 32;
          const uint32_t qo = (kk >> 2) * (PT_N * 128) + (kk & 3) * 32;
          umma_f16_ss(d, make_smem_desc_sw128(sK + ko, 16, 1024), make_smem_desc_sw128(sQ + qo, 16, 1024),
                      idesc_qk, kk > 0 ? 1u : 0u);
        }
        umma_commit(bar(S_FULL + (t & 1)));
      };
      bool ok = mbar_wait(bar(KV_FULL + 0), 0, abort_word, FT_ERR_TIMEOUT_MMA);
      if (ok) {
        tc_fence_after();
        issue_qk(0);
      }
      for (int t = 0; t < n_tiles && ok; ++t) {
        if (t + 1 < n_tiles) {
          // S buffer (t+1)&1 was last read by the softmax of tile t-1, which has arrived on P_FULL
          ok = mbar_wait(bar(KV_FULL + (t + 1) % PT_STAGES), ((t + 1) / PT_STAGES) & 1, abort_word, FT_ERR_TIMEOUT_MMA);
          if (!ok) break;
          tc_fence_after();
          issue_qk(t + 1);
        }
        const int st = t % PT_STAGES;
        ok = mbar_wait(bar(P_FULL + (t & 1)), (t >> 1) & 1, abort_word, FT_ERR_TIMEOUT_MMA);
        if (!ok) break;
        tc_fence_after();
        const uint32_t sV = sbase + st * Cfg::STAGE_BYTES + Cfg::K_BYTES;
        const uint32_t pb = sP + (t & 1) * Cfg::P_BYTES;
#pragma unroll
        for (int kk = 0; kk < PT_TILE / 16; ++kk) {
          // A = V^T: 16 keys = 2048 bytes down each 64-wide chunk, chunks CHUNK bytes apart
          umma_f16_ss(tmem_base + COL_O, make_smem_desc_sw128(sV + kk * 2048, Cfg::CHUNK, 1024),
                      make_smem_desc_sw128(pb + (kk >> 2) * (PT_N * 128) + (kk & 3) * 32, 16, 1024), idesc_pv,
                      (t > 0 || kk > 0) ? 1u : 0u);
        }
        umma_commit(bar(O_DONE));
        umma_commit(bar(ST_EMPTY + st));
      }
    }
  } else if (warp >= 4 && warp < 8) {
    // ------------------------------------------------------------------ softmax / epilogue
    const int ew = warp & 3;
    const int r = ew * 32 + lane;   // key of the tile while scoring, output dim in the epilogue
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(ew * 32) << 16);
    float m_ref[G], l_part[G], slope[G];
#pragma unroll
    for (int g = 0; g < G; ++g) {
      m_ref[g] = -INFINITY;
      l_part[g] = 0.f;
      slope[g] = slopes && g < g_real ? slopes[kvh * g_real + g] * ATT_LOG2E : 0.f;
    }
    bool ok = true;
    // Every softmax thread runs every iteration down to the named barriers, also after a failed
    // wait (later waits then fail at once), so no barrier is ever left short of arrivals.
    for (int t = 0; t < n_tiles; ++t) {
      const int sb = t & 1;
      if (ok && !mbar_wait(bar(S_FULL + sb), (t >> 1) & 1, abort_word, FT_ERR_TIMEOUT_EPILOGUE)) ok = false;
      uint32_t sv[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) sv[i] = 0u;
      if (ok) {
        tc_fence_after();
        tmem_ld_32x16(lane_addr + COL_S + sb * PT_N, sv);
        tmem_ld_wait();
      }
      const bool is_pool = tile_lo + t < pool_tiles;
      const int key = (tile_lo + t + (is_pool ? 0 : key_tile)) * PT_TILE + r;
      const bool valid = is_pool ? key < n_pool : key < len && key >= first;
      float s[G], mx[G];
#pragma unroll
      for (int g = 0; g < G; ++g) {
        s[g] = valid ? __uint_as_float(sv[g]) * scale_log2 - slope[g] * static_cast<float>(len - 1 - key) : -INFINITY;
        mx[g] = warp_max(s[g]);
      }
      if (lane == 0) {
#pragma unroll
        for (int g = 0; g < G; ++g) s_red[ew * PT_N + g] = mx[g];
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      float alpha[G];
      bool any_rescale = false;
#pragma unroll
      for (int g = 0; g < G; ++g) {
        const float tile_max = fmaxf(fmaxf(s_red[g], s_red[PT_N + g]), fmaxf(s_red[2 * PT_N + g], s_red[3 * PT_N + g]));
        alpha[g] = 1.f;
        if (tile_max > m_ref[g] + PT_RESCALE) {   // the same decision in every thread
          alpha[g] = fast_exp2(m_ref[g] - tile_max);  // m_ref = -inf on the first tile -> 0
          m_ref[g] = tile_max;
          any_rescale = true;
        }
        l_part[g] *= alpha[g];
      }
      // O of the earlier tiles (and the P buffer of tile t-2) are free once PV(t-1) has completed
      if (t > 0 && ok && !mbar_wait(bar(O_DONE), (t - 1) & 1, abort_word, FT_ERR_TIMEOUT_EPILOGUE)) ok = false;
      if (t > 0 && any_rescale && ok) {
        tc_fence_after();
        uint32_t ov[16];
        tmem_ld_32x16(lane_addr + COL_O, ov);   // this thread's output dim, one column per head
        tmem_ld_wait();
#pragma unroll
        for (int g = 0; g < G; ++g) ov[g] = __float_as_uint(__uint_as_float(ov[g]) * alpha[g]);
        tmem_st_32x16(lane_addr + COL_O, ov);
        tmem_st_wait();
      }
      // P^T[head g][key r] as bf16 into the K-major operand tile (rows >= G stay zero)
      {
        uint8_t* pb = smem + Cfg::OFF_P + sb * Cfg::P_BYTES + (r >> 6) * (PT_N * 128);
        const int kc = r & 63;
#pragma unroll
        for (int g = 0; g < G; ++g) {
          const float pv = valid ? fast_exp2(s[g] - m_ref[g]) : 0.f;
          const __nv_bfloat16 pb16 = __float2bfloat16(pv);
          l_part[g] += __bfloat162float(pb16);   // the sum of what the MMA will actually use
          *reinterpret_cast<__nv_bfloat16*>(pb + g * 128 + (((kc >> 3) ^ (g & 7)) << 4) + (kc & 7) * 2) = pb16;
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (ok && lane == 0) mbar_arrive(bar(P_FULL + sb));
      // s_red is rewritten in the next iteration: every thread must have read it
      asm volatile("bar.sync 1, 128;" ::: "memory");
    }
    if (ok && n_tiles > 0) {
      ok = mbar_wait(bar(O_DONE), (n_tiles - 1) & 1, abort_word, FT_ERR_TIMEOUT_EPILOGUE);
      tc_fence_after();
    }
    // total l per head: sum of the per-thread partial sums
    float l_tot[G];
#pragma unroll
    for (int g = 0; g < G; ++g) {
      const float ws = warp_sum(l_part[g]);
      if (lane == 0) s_red[ew * PT_N + g] = ws;
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
#pragma unroll
    for (int g = 0; g < G; ++g) l_tot[g] = s_red[g] + s_red[PT_N + g] + s_red[2 * PT_N + g] + s_red[3 * PT_N + g];
    if (ok) {                                     // whole warps: the TMEM load is a warp-wide instruction
      uint32_t ov[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) ov[i] = 0u;
      if (n_tiles > 0) {
        tmem_ld_32x16(lane_addr + COL_O, ov);
        tmem_ld_wait();
      }
#pragma unroll
      for (int g = 0; g < G; ++g) {
        if (g >= g_real || r >= Dv) continue;
        const int hq = kvh * g_real + g;
        const float acc = __uint_as_float(ov[g]);
        if (n_splits == 1) {
          float mm = m_ref[g], ll = l_tot[g], o = acc;
          sink_join(sink, hq, mm, ll, o);
          out[static_cast<long long>(b) * ldo + static_cast<long long>(hq) * Dv + r] =
              __float2bfloat16(ll > 0.f ? o / ll * out_scale * head_gate_bf16(gate, b, hq, r) : 0.f);
        } else {
          const long long pidx = (static_cast<long long>(b) * Hq + hq) * n_splits + split;
          part_o[pidx * Dv + r] = acc;
          if (r == 0) { part_ml[pidx * 2] = m_ref[g]; part_ml[pidx * 2 + 1] = l_tot[g]; }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 2) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 64);
  }
  if (threadIdx.x == 0 && *abort_word != 0 && status) atomicCAS(status, 0, *abort_word);
}

// ----------------------------------------------------------------------------- any rows, any sizes
// Row i attends to keys 0 .. visible[i] - 1 of sequence row_slot[i] (the last `window` of them).  A CTA owns one row and up to
// PR_HEADS query heads of one KV head; its four warps walk tiles of 32 keys (lane = key while scoring,
// lane = value dim while accumulating) with an fp32 online softmax each, merged at the end.
constexpr int PR_HEADS = 8;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void from_f32(float v, float* p) { *p = v; }
__device__ __forceinline__ void from_f32(float v, __nv_bfloat16* p) { *p = __float2bfloat16(v); }

template <typename T>
__global__ void __launch_bounds__(PD_THREADS)
paged_rows_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                  const int* __restrict__ block_table, const int* __restrict__ row_slot, const int* __restrict__ visible,
                  HeadGate gate, T* __restrict__ out, int rows, int Hq, int Hkv, int D, int Dv, long long ldq, long long ldo,
                  int ldv, int block_size, int max_blocks, int num_blocks, float scale, KeyRange range, PooledKeys pooled,
                  const float* __restrict__ slopes, const float* __restrict__ sink, float out_scale, int head_groups) {
  extern __shared__ float sm[];
  const int g_all = Hq / Hkv;
  const int kvh = blockIdx.y / head_groups, h0 = (blockIdx.y % head_groups) * PR_HEADS;
  const int g = min(PR_HEADS, g_all - h0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* s_q = sm;                                   // [g][D], scaled by scale * log2(e)
  float* s_o = s_q + PR_HEADS * D;                   // [warps][g][Dv]
  float* s_p = s_o + PD_WARPS * PR_HEADS * Dv;       // [warps][g][32]
  float* s_m = s_p + PD_WARPS * PR_HEADS * 32;       // [warps][g]
  float* s_l = s_m + PD_WARPS * PR_HEADS;
  for (int row = blockIdx.x; row < rows; row += gridDim.x) {
    __syncthreads();
    const int len = min(visible[row], max_blocks * block_size);
    const int first = range.first_visible(len);
    const int* bt = block_table + static_cast<long long>(row_slot[row]) * max_blocks;
    for (int i = threadIdx.x; i < g * D; i += PD_THREADS) {
      const int h = i / D, d = i - h * D;
      s_q[h * D + d] = to_f32(q[static_cast<long long>(row) * ldq + static_cast<long long>(kvh * g_all + h0 + h) * D + d]) *
                       (scale * 1.4426950408889634f);
    }
    for (int i = threadIdx.x; i < PD_WARPS * PR_HEADS * Dv; i += PD_THREADS) s_o[i] = 0.f;
    float m[PR_HEADS], l[PR_HEADS];
#pragma unroll
    for (int h = 0; h < PR_HEADS; ++h) { m[h] = -INFINITY; l[h] = 0.f; }
    __syncthreads();
    // tiles of 32 pooled blocks, then tiles of 32 keys
    const int n_pool = pooled.count(first), pool_tiles = (n_pool + 31) / 32, tiles = pool_tiles + max(0, (len - first / 32 * 32 + 31) / 32);
    auto key_row = [&](int kk) {
      const int blk = min(max(bt[kk / block_size], 0), num_blocks - 1);
      return static_cast<long long>(blk) * block_size + kk % block_size;
    };
    for (int tile = warp; tile < tiles; tile += PD_WARPS) {
      const bool is_pool = tile < pool_tiles;
      const int key0 = is_pool ? tile * 32 : (first / 32 + tile - pool_tiles) * 32, end = is_pool ? n_pool : len;
      const int key = key0 + lane;
      const bool valid = key < end && (is_pool || key >= first);
      const int kk = key < end ? key : key0;
      const T* kr = is_pool ? static_cast<const T*>(pooled.k) + (pooled.row(kk, bt, block_size, max_blocks, num_blocks) * Hkv + kvh) * D
                            : k_cache + (key_row(kk) * Hkv + kvh) * D;
      float s[PR_HEADS];
#pragma unroll
      for (int h = 0; h < PR_HEADS; ++h) s[h] = 0.f;
      for (int d = 0; d < D; ++d) {
        const float kd = to_f32(kr[d]);
#pragma unroll
        for (int h = 0; h < PR_HEADS; ++h)
          if (h < g) s[h] += kd * s_q[h * D + d];
      }
      float* o = s_o + warp * PR_HEADS * Dv;
      float* pr = s_p + warp * PR_HEADS * 32;
      float alpha[PR_HEADS];
#pragma unroll
      for (int h = 0; h < PR_HEADS; ++h) {
        alpha[h] = 1.f;
        if (h >= g) continue;
        const float bias = slopes ? slopes[kvh * g_all + h0 + h] * ATT_LOG2E * static_cast<float>(len - 1 - key) : 0.f;
        const float sv = valid ? s[h] - bias : -INFINITY;
        const float m_new = fmaxf(m[h], warp_max(sv));
        const float pv = valid ? exp2f(sv - m_new) : 0.f;
        alpha[h] = exp2f(m[h] - m_new);              // first tile: exp2(-inf) = 0
        l[h] = l[h] * alpha[h] + warp_sum(pv);
        m[h] = m_new;
        pr[h * 32 + lane] = pv;
      }
      __syncwarp();
      const int n_keys = min(32, end - key0);
      for (int d = lane; d < Dv; d += 32) {
        float acc[PR_HEADS];
#pragma unroll
        for (int h = 0; h < PR_HEADS; ++h) acc[h] = h < g ? o[h * Dv + d] * alpha[h] : 0.f;
        for (int j = 0; j < n_keys; ++j) {
          const float vd = is_pool ? to_f32(static_cast<const T*>(pooled.v)[(pooled.row(key0 + j, bt, block_size, max_blocks, num_blocks) * Hkv + kvh) * Dv + d])
                                   : to_f32(v_cache[(key_row(key0 + j) * Hkv + kvh) * ldv + d]);
#pragma unroll
          for (int h = 0; h < PR_HEADS; ++h)
            if (h < g) acc[h] += pr[h * 32 + j] * vd;
        }
#pragma unroll
        for (int h = 0; h < PR_HEADS; ++h)
          if (h < g) o[h * Dv + d] = acc[h];
      }
      __syncwarp();
    }
    if (lane == 0) {
#pragma unroll
      for (int h = 0; h < PR_HEADS; ++h)
        if (h < g) { s_m[warp * PR_HEADS + h] = m[h]; s_l[warp * PR_HEADS + h] = l[h]; }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < g * Dv; i += PD_THREADS) {
      const int h = i / Dv, d = i - h * Dv;
      float mm = -INFINITY;
#pragma unroll
      for (int w = 0; w < PD_WARPS; ++w) mm = fmaxf(mm, s_m[w * PR_HEADS + h]);
      float ll = 0.f, acc = 0.f;
#pragma unroll
      for (int w = 0; w < PD_WARPS; ++w) {
        const float mw = s_m[w * PR_HEADS + h];
        const float sc = mw == -INFINITY ? 0.f : exp2f(mw - mm);
        ll += s_l[w * PR_HEADS + h] * sc;
        acc += s_o[(w * PR_HEADS + h) * Dv + d] * sc;
      }
      const int hq = kvh * g_all + h0 + h;
      sink_join(sink, hq, mm, ll, acc);
      float v = ll > 0.f ? acc / ll * out_scale : 0.f;
      if (gate.g) v *= gate_value(to_f32(static_cast<const T*>(gate.g)[gate.at(row, hq, d)]));
      from_f32(v, out + static_cast<long long>(row) * ldo + static_cast<long long>(hq) * Dv + d);
    }
  }
}

}  // namespace ft

using namespace ft;

// Append keys [T, Hkv, D] and values [T, Hkv, Dv] of elem_bytes-sized elements (2 or 4; strides in elements).
FT_API int ft_kv_append(const void* k_new, const void* v_new, void* k_cache, void* v_cache, const int* block_table,
                        const int* pos, const int* seq_ids, int T, int tokens_per_seq, int Hkv, int D, int Dv, int elem_bytes,
                        long long ldk, long long ldv, int block_size, int max_blocks, int num_blocks,
                        int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(k_new && v_new && k_cache && v_cache && block_table && pos, "ft_kv_append: null pointer");
  FT_REQUIRE(elem_bytes == 2 || elem_bytes == 4, "ft_kv_append: element size %d", elem_bytes);
  const int unit = 16 / elem_bytes;
  FT_REQUIRE((Hkv * D) % unit == 0 && (Hkv * Dv) % unit == 0 && ldk % unit == 0 && ldv % unit == 0 && block_size > 0 &&
                 (seq_ids || tokens_per_seq > 0), "ft_kv_append: bad layout");
  FT_REQUIRE(((reinterpret_cast<uintptr_t>(k_new) | reinterpret_cast<uintptr_t>(v_new) | reinterpret_cast<uintptr_t>(k_cache) |
               reinterpret_cast<uintptr_t>(v_cache)) & 15) == 0, "ft_kv_append: pointers must be 16-byte aligned");
  if (T <= 0) return FT_E_OK;
  const int grid = T < sm_count(device) * 8 ? T : sm_count(device) * 8;
  kv_append_kernel<<<grid, 128, 0, stream>>>(static_cast<const uint4*>(k_new), static_cast<const uint4*>(v_new),
                                             static_cast<uint4*>(k_cache), static_cast<uint4*>(v_cache), block_table, pos,
                                             seq_ids, T, tokens_per_seq, Hkv * D / unit, Hkv * Dv / unit, ldk / unit, ldv / unit,
                                             block_size, max_blocks, num_blocks);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// Means of whole blocks of keys and values.  Block b of a sequence holds its positions b * pool .. b * pool + pool - 1 and lies with the
// page of its last position: k_pool [num_blocks, (block_size - 1) / pool + 1, Hkv, D], place b - page * block_size / pool (v_pool
// likewise).  For every one of `rows` rows (positions pos of sequences slots, already in the cache) that ends a block the means
// are formed in fp32.  bf16, or fp32 with f32; head sizes such that a token's keys and values are whole 8-element vectors.
FT_API int ft_pool_blocks(const void* k_cache, const void* v_cache, void* k_pool, void* v_pool, const int* block_table, const int* pos,
                          const int* slots, int rows, int Hkv, int D, int Dv, int pool, int f32, int block_size, int max_blocks, int num_blocks,
                          int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(k_cache && v_cache && k_pool && v_pool && block_table && pos && slots, "ft_pool_blocks: null pointer");
  FT_REQUIRE(Hkv > 0 && D > 0 && Dv > 0 && (Hkv * D) % 8 == 0 && (Hkv * Dv) % 8 == 0 && pool > 0 && block_size > 0 && max_blocks > 0 && num_blocks > 0,
             "ft_pool_blocks: %d heads of %d / %d, blocks of %d", Hkv, D, Dv, pool);
  FT_REQUIRE(((reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) | reinterpret_cast<uintptr_t>(k_pool) |
               reinterpret_cast<uintptr_t>(v_pool)) & 15) == 0, "ft_pool_blocks: pointers must be 16-byte aligned");
  if (rows <= 0) return FT_E_OK;
  const int kw = Hkv * D, vw = Hkv * Dv, per_page = (block_size - 1) / pool + 1;
  const int parts = (kw + vw + PB_THREADS * 8 - 1) / (PB_THREADS * 8);
  // enough CTAs for the GPU at once, up to a warp's worth of rows each
  int walk = rows / (sm_count(device) * 3);
  walk = walk < 1 ? 1 : (walk > 32 ? 32 : walk);
  const dim3 grid((rows + walk - 1) / walk, parts);
#define FT_PB(T) \
  pool_blocks_kernel<T><<<grid, PB_THREADS, 0, stream>>>(static_cast<const T*>(k_cache), static_cast<const T*>(v_cache), static_cast<T*>(k_pool), \
      static_cast<T*>(v_pool), block_table, pos, slots, rows, walk, kw, vw, pool, per_page, block_size, max_blocks, num_blocks)
  if (f32) FT_PB(float); else FT_PB(__nv_bfloat16);
#undef FT_PB
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// Scratch floats needed for n_splits > 1: B * Hq * n_splits * (Dv + 2).
FT_API long long ft_paged_decode_scratch(int B, int Hq, int Dv, int n_splits) {
  return n_splits > 1 ? static_cast<long long>(B) * Hq * n_splits * (Dv + 2) : 0;
}

// q: [B, Hq, D] (row stride ldq), out: [B, Hq, Dv] (row stride ldo), ctx_len: int32 [B] = number of
// cached tokens to attend to (including the current one, which must already be appended), of which the last
// `window` are visible (0: all), or those of the row's own chunk of `chunk` positions (0: all).  slopes (fp32 [Hq] or null): a
// head's slope times the distance of a key is taken off its score.  The result is multiplied by out_scale.  Row b reads sequence row_slot[b] of the block table (null: sequence b).  sink
// (fp32 [Hq] or null): exp(sink) joins a head's denominator.  gate (bf16 or null): element d of head h of row b is
// multiplied by sigmoid(gate[b * ldg + h * gate_head + d * gate_elem]); one number per head with gate_elem 0.  pool (with a window, without
// chunk and slopes; 0: none): the row also sees k_pool and v_pool (see ft_pool_blocks) of the blocks wholly ahead of its window.
FT_API int ft_paged_decode(const void* q, const void* k_cache, const void* v_cache, const int* block_table,
                           const int* row_slot, const int* ctx_len, const void* gate, const float* sink, void* out,
                           float* scratch, int B, int Hq, int Hkv, int D, int Dv, long long ldq, long long ldg,
                           int gate_head, int gate_elem, long long ldo, int block_size, int max_blocks, int num_blocks,
                           float scale, int window, int chunk, const void* k_pool, const void* v_pool, int pool, const float* slopes,
                           float out_scale, int n_splits, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(q && k_cache && v_cache && block_table && ctx_len && out, "ft_paged_decode: null pointer");
  FT_REQUIRE(B >= 0 && Hkv > 0 && Hq > 0 && Hq % Hkv == 0 && block_size > 0 && max_blocks > 0 && num_blocks > 0, "ft_paged_decode: bad shape");
  FT_REQUIRE(window >= 0 && chunk >= 0, "ft_paged_decode: negative window or chunk");
  FT_REQUIRE(pool == 0 || (pool > 0 && window > 0 && !chunk && !slopes && k_pool && v_pool), "ft_paged_decode: blocks of %d keys", pool);
  const PooledKeys pooled = pooled_keys(k_pool, v_pool, pool, block_size);
  const KeyRange range = {window, chunk};
  FT_REQUIRE(n_splits >= 1 && (n_splits == 1 || scratch), "ft_paged_decode: splits need scratch");
  if (B == 0) return FT_E_OK;
  const float sl2 = scale * 1.4426950408889634f;
  float* part_o = scratch;
  float* part_ml = scratch ? scratch + static_cast<long long>(B) * Hq * n_splits * Dv : nullptr;
  dim3 grid(n_splits, Hkv, B);
  const int G = Hq / Hkv;
  const HeadGate hg = {gate, ldg, gate_head, gate_elem};
  // equal head sizes of 64 half fill the tensor-core kernel's value tile: the CUDA-core kernel is faster there
  // (127 against 156 us at 64 rows x 2048 keys x 8 KV heads) and keeps P in fp32
  const bool core64 = pool == 0 && D == 64 && Dv == 64 && (G == 1 || G == 2 || G == 4 || G == 8) &&
                      ((reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache)) & 15) == 0;
  const bool tensor_core = !core64 && D >= 16 && D <= 128 && D % 16 == 0 && Dv >= 16 && Dv <= 128 && Dv % 16 == 0 && G <= PT_N &&
                           (reinterpret_cast<uintptr_t>(q) & 15) == 0 && ldq % 8 == 0 &&
                           ((reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache)) & 15) == 0;
  if (tensor_core) {
    int* status = device_status_word(device);
#define FT_PT_LAUNCH(HH, GG)                                                                                    \
  {                                                                                                             \
    auto kern = paged_decode_tc_kernel<HH, GG>;                                                                 \
    static bool attr_set[64] = {false};                                                                         \
    if (!attr_set[device]) {                                                                                    \
      FT_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, PtCfg<HH>::SMEM_BYTES)); \
      attr_set[device] = true;                                                                                  \
    }                                                                                                           \
    kern<<<grid, PT_THREADS, PtCfg<HH>::SMEM_BYTES, stream>>>(                                                  \
        static_cast<const __nv_bfloat16*>(k_cache), static_cast<const __nv_bfloat16*>(v_cache),                \
        static_cast<const __nv_bfloat16*>(q), block_table, row_slot, ctx_len, static_cast<__nv_bfloat16*>(out), \
        part_o, part_ml, Hq, Hkv, D, Dv, G, ldq, ldo, block_size, max_blocks, num_blocks, sl2, n_splits, range, pooled, slopes, sink, hg, out_scale, status); \
  }
#define FT_PT_BY_G(HH)                     \
  if (G == 1) FT_PT_LAUNCH(HH, 1)          \
  else if (G == 2) FT_PT_LAUNCH(HH, 2)     \
  else if (G <= 4) FT_PT_LAUNCH(HH, 4)     \
  else if (G <= 8) FT_PT_LAUNCH(HH, 8)     \
  else FT_PT_LAUNCH(HH, 16)
    if (D > 64) { FT_PT_BY_G(128) } else { FT_PT_BY_G(64) }
#undef FT_PT_BY_G
#undef FT_PT_LAUNCH
  } else {
    FT_REQUIRE(pool == 0, "ft_paged_decode: blocks of keys need head sizes that are multiples of 16 up to 128, 16-byte aligned rows");
    FT_REQUIRE((D == 64 || D == 128) && D == Dv, "ft_paged_decode: head sizes %d / %d not supported (multiples of 16 up to 128, 16-byte aligned rows)", D, Dv);
#define FT_PD_LAUNCH(DD, GG)                                                                                   \
  paged_decode_kernel<DD, GG><<<grid, PD_THREADS, 0, stream>>>(                                                \
      static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(k_cache),                        \
      static_cast<const __nv_bfloat16*>(v_cache), block_table, row_slot, ctx_len, static_cast<__nv_bfloat16*>(out), \
      part_o, part_ml, Hq, Hkv, ldq, ldo, block_size, max_blocks, num_blocks, sl2, n_splits, range, slopes, sink, hg, out_scale)
#define FT_PD_BY_G(DD)                                             \
  switch (G) {                                                     \
    case 1: FT_PD_LAUNCH(DD, 1); break;                            \
    case 2: FT_PD_LAUNCH(DD, 2); break;                            \
    case 4: FT_PD_LAUNCH(DD, 4); break;                            \
    case 8: FT_PD_LAUNCH(DD, 8); break;                            \
    default:                                                       \
      set_last_error("ft_paged_decode: group size %d not supported (1, 2, 4, 8)", G); \
      return FT_E_BAD_ARG;                                         \
  }
    if (D == 128) { FT_PD_BY_G(128) } else { FT_PD_BY_G(64) }
#undef FT_PD_BY_G
#undef FT_PD_LAUNCH
  }
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  if (n_splits > 1) {
    dim3 g2(Hq, B);
    paged_decode_combine_kernel<<<g2, Dv <= 64 ? 64 : 128, 0, stream>>>(part_o, part_ml, static_cast<__nv_bfloat16*>(out), Hq, Dv, ldo, n_splits, sink, hg, out_scale);
    FT_CUDA_CHECK(cudaGetLastError());
    count_launch();
  }
  return FT_E_OK;
}

// Attention of arbitrary rows over the paged cache (see paged_rows_kernel): q [rows, Hq, D], out
// [rows, Hq, Dv], row_slot / visible int32 [rows]; window, chunk, pool, slopes, sink (always fp32) and gate as in
// ft_paged_decode.  A cached value has Dv elements, the next head's begins ldv later (values that are the leading elements of
// the keys: v_cache = k_cache, ldv = D).  All other tensors bf16, or fp32 with f32.
FT_API int ft_paged_rows(const void* q, const void* k_cache, const void* v_cache, const int* block_table, const int* row_slot,
                         const int* visible, const void* gate, const float* sink, void* out, int rows, int Hq, int Hkv,
                         int D, int Dv, long long ldq, long long ldg, int gate_head, int gate_elem, long long ldo,
                         int ldv, int block_size, int max_blocks, int num_blocks, float scale, int window, int chunk,
                         const void* k_pool, const void* v_pool, int pool, const float* slopes, float out_scale, int f32, int device,
                         cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(q && k_cache && v_cache && block_table && row_slot && visible && out, "ft_paged_rows: null pointer");
  FT_REQUIRE(Hkv > 0 && Hq > 0 && Hq % Hkv == 0 && D > 0 && Dv > 0 && block_size > 0 && max_blocks > 0 && num_blocks > 0 && window >= 0 && chunk >= 0 && ldv >= Dv, "ft_paged_rows: bad shape");
  FT_REQUIRE(pool == 0 || (pool > 0 && window > 0 && !chunk && !slopes && k_pool && v_pool), "ft_paged_rows: blocks of %d keys", pool);
  if (rows <= 0) return FT_E_OK;
  const int groups = (Hq / Hkv + PR_HEADS - 1) / PR_HEADS;
  const size_t smem = sizeof(float) * (static_cast<size_t>(PR_HEADS) * D + static_cast<size_t>(PD_WARPS) * PR_HEADS * Dv +
                                       PD_WARPS * PR_HEADS * 32 + 2 * PD_WARPS * PR_HEADS);
  FT_REQUIRE(smem <= 200 * 1024 && static_cast<long long>(Hkv) * groups < 65536, "ft_paged_rows: head sizes %d / %d are too large", D, Dv);
  const dim3 grid(rows < 65536 ? rows : 65536, Hkv * groups);
  const HeadGate hg = {gate, ldg, gate_head, gate_elem};
#define FT_PR_LAUNCH(T)                                                                                                      \
  {                                                                                                                          \
    FT_CUDA_CHECK(cudaFuncSetAttribute(paged_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem))); \
    paged_rows_kernel<T><<<grid, PD_THREADS, smem, stream>>>(static_cast<const T*>(q), static_cast<const T*>(k_cache),       \
        static_cast<const T*>(v_cache), block_table, row_slot, visible, hg, static_cast<T*>(out), rows, Hq, Hkv, D, Dv, ldq, \
        ldo, ldv, block_size, max_blocks, num_blocks, scale, KeyRange{window, chunk}, pooled_keys(k_pool, v_pool, pool, block_size), slopes, sink, out_scale, groups); \
  }
  if (f32) FT_PR_LAUNCH(float) else FT_PR_LAUNCH(__nv_bfloat16)
#undef FT_PR_LAUNCH
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}
