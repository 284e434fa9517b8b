// Grouped matrix products on tcgen05 / TMEM: many small problems with weights of their own in one launch.
//
//   out[rows of group g, n] = epilogue( sum_k A[row, k (+ g * a_col)] * W[g][part][n, k] )
//
// W is [groups, parts, N, K] (bf16, K-major).  With two parts a tile accumulates both products of the same rows, so
// that the epilogue can combine them:
//   EPI_STORE  one part:  C = sum, optionally the square of its relu, or times the sigmoid of a gate per element
//   EPI_GLU    two parts: C = act(r sum_0) * (r sum_1), r a factor per row (a routed token's weight: scaling the
//              two sums is scaling the input)
//   EPI_RGLRU  two parts: the gates of a real-gated linear recurrence (see recurrent.cuh), recurrence and all for
//              rows that are a sequence's only token, decay and input term for the others
//
// Groups are either segments of rows (a mixture of experts: rows sorted by expert, segments listed on the device by
// moe_build_kernel, so that no launch depends on the host knowing the counts) or blocks of columns (a block-diagonal
// matrix: every row takes part in every group with its own columns, and the results of group g begin at column g * out_col).
//
// The kernel is persistent, one CTA per SM, 384 threads (EPI_RGLRU: 640):
//   warp 0     TMA producer: a ring of {A 128 x 64, W BN x 64} tiles; the A box has only as many rows as the caller
//              says a segment can have (a decode step: 16 or 32), so small batches move little besides weights
//   warp 1     MMA issuer
//   warp 2     TMEM allocator (two accumulators of BN columns)
//   warps 4-   epilogue, two warpgroups that share a tile's columns (EPI_RGLRU: four, its arithmetic is the bound)
// Rows of a tile past the end of its segment hold other rows or stale shared memory; rows of an MMA are independent
// and those are not stored.  All waits are bounded and report through the device status word.
//
// fp32 problems run on a plain tiled kernel with the same groups and epilogues.
#include <initializer_list>

#include "recurrent.cuh"
#include "row_vec.cuh"

namespace ft {

constexpr int GG_BM = 128;
constexpr int GG_BK = 64;
constexpr int GG_GROUP_M = 16;

enum : int { EPI_STORE = 0, EPI_GLU = 1, EPI_RGLRU = 2 };
constexpr int GG_RELU2 = 3;

struct GroupedParams {
  // segments: items[3 i ..] = group, first row, rows; n_items_dev on the device.  Column blocks: items null,
  // every group has `rows` rows.
  const int* items;
  const int* n_items_dev;
  int max_items, rows, groups, a_col, a_rows;
  int N, K, parts;
  void* out;                 // EPI_STORE / EPI_GLU: [rows, ldo]
  long long ldo;
  int out_col;
  const void* gate;          // EPI_STORE: element (row, column) is multiplied by sigmoid(gate[row * ldgate + column]); null: not
  long long ldgate;
  const float* row_scale;    // EPI_GLU: per row, or null
  int act;                   // EPI_GLU: of the first sum; EPI_STORE: GG_RELU2 or 0
  RglruGateParams gates;     // EPI_RGLRU
  int* status;
};

struct GroupedTile {
  int group, row0, rows, n0;
};

// Tile `t`: neighbouring tiles share weights over up to GG_GROUP_M row blocks, then move to the next columns.
__device__ __forceinline__ GroupedTile grouped_tile(const GroupedParams& p, int t, int m_items, int n_blocks, int n_width) {
  const int span = GG_GROUP_M * n_blocks;
  const int g = t / span, first = g * GG_GROUP_M;
  const int gm = min(GG_GROUP_M, m_items - first);
  const int r = t - g * span;
  const int item = first + r % gm;
  GroupedTile out;
  out.n0 = (r / gm) * n_width;
  if (p.items) {
    out.group = p.items[3 * item];
    out.row0 = p.items[3 * item + 1];
    out.rows = p.items[3 * item + 2];
  } else {
    const int per = (p.rows + GG_BM - 1) / GG_BM;
    out.group = item / per;
    out.row0 = (item - out.group * per) * GG_BM;
    out.rows = min(GG_BM, p.rows - out.row0);
  }
  return out;
}

__device__ __forceinline__ int grouped_items(const GroupedParams& p) {
  if (p.items) return min(*p.n_items_dev, p.max_items);
  return p.groups * ((p.rows + GG_BM - 1) / GG_BM);
}

__device__ __forceinline__ float glu_act(float g, int act) {
  if (act == 1) return fmaxf(g, 0.f);
  if (act == 2) {
    const float k = 0.7978845608028654f * (g + 0.044715f * g * g * g);
    return 0.5f * g * (1.f + tanhf(k));
  }
  return __fdividef(g, 1.f + __expf(-g));
}

template <int BN, int EPI>
struct GgCfg {
  static constexpr int EPI_WARPS = EPI == EPI_RGLRU ? 16 : 8;
  static constexpr int THREADS = 128 + 32 * EPI_WARPS;
  static constexpr int A_BYTES = GG_BM * GG_BK * 2;
  static constexpr int B_BYTES = BN * GG_BK * 2;
  static constexpr int STAGE_BYTES = A_BYTES + B_BYTES;
  static constexpr int STAGES = (216 * 1024) / STAGE_BYTES > 6 ? 6 : (216 * 1024) / STAGE_BYTES;
  static constexpr int TMEM_COLS = 2 * BN;
  static constexpr int SMEM_BYTES = STAGES * STAGE_BYTES + 1024 + 256;
};

template <int BN, int EPI>
__global__ void __launch_bounds__(GgCfg<BN, EPI>::THREADS, 1)
grouped_gemm_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB, const GroupedParams p) {
  using Cfg = GgCfg<BN, EPI>;
  constexpr int STAGES = Cfg::STAGES;
  constexpr int NW = EPI == EPI_STORE ? BN : BN / 2;    // output columns of a tile
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + STAGES * Cfg::STAGE_BYTES);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * STAGES + 4);
  volatile int* abort_word = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t smem_base = smem_u32(smem), bar_base = smem_u32(bars);
  auto full_bar = [&](int s) { return bar_base + 8u * s; };
  auto empty_bar = [&](int s) { return bar_base + 8u * (STAGES + s); };
  auto tfull_bar = [&](int a) { return bar_base + 8u * (2 * STAGES + a); };
  auto tempty_bar = [&](int a) { return bar_base + 8u * (2 * STAGES + 2 + a); };

  if (threadIdx.x == 0) {
    *abort_word = 0;
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(full_bar(s), 1);
      mbar_init(empty_bar(s), 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(tfull_bar(a), 1);
      mbar_init(tempty_bar(a), Cfg::EPI_WARPS);   // one arrival per epilogue warp
    }
    fence_mbar_init();
    tma_prefetch_desc(&tmA);
    tma_prefetch_desc(&tmB);
  }
  if (warp == 2) {
    tmem_alloc(smem_u32(tmem_slot), Cfg::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const int m_items = grouped_items(p);
  const int n_blocks = (p.N + NW - 1) / NW;
  const int num_tiles = m_items * n_blocks;
  const int k_blocks = (p.K + GG_BK - 1) / GG_BK;

  if (warp == 0) {
    if (lane == 0) {
      int stage = 0;
      uint32_t phase = 0;
      bool ok = true;
      const uint32_t bytes = static_cast<uint32_t>(p.a_rows) * (GG_BK * 2) + Cfg::B_BYTES;
      for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
        const GroupedTile t = grouped_tile(p, tile, m_items, n_blocks, NW);
        const int b0 = t.group * p.parts * p.N + t.n0;                        // W row of the first half of the tile
        const int b1 = b0 + (EPI == EPI_STORE ? BN / 2 : p.N);
        for (int kb = 0; kb < k_blocks; ++kb) {
          if (!mbar_wait(empty_bar(stage), phase ^ 1u, abort_word, FT_ERR_TIMEOUT_PRODUCER)) { ok = false; break; }
          const uint32_t sA = smem_base + stage * Cfg::STAGE_BYTES, sB = sA + Cfg::A_BYTES;
          mbar_expect_tx(full_bar(stage), bytes);
          tma_load_2d(sA, &tmA, full_bar(stage), kb * GG_BK + t.group * p.a_col, t.row0);
          tma_load_2d(sB, &tmB, full_bar(stage), kb * GG_BK, b0);
          tma_load_2d(sB + Cfg::B_BYTES / 2, &tmB, full_bar(stage), kb * GG_BK, b1);
          if (++stage == STAGES) { stage = 0; phase ^= 1u; }
        }
      }
      if (!ok) {   // let copies in flight land before the CTA leaves
        const unsigned long long t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc_f16(GG_BM, BN, 1, 0, 0);
      int stage = 0, acc = 0;
      uint32_t phase = 0, acc_phase = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
        if (!mbar_wait(tempty_bar(acc), acc_phase ^ 1u, abort_word, FT_ERR_TIMEOUT_MMA)) break;
        tc_fence_after();
        const uint32_t d_tmem = tmem_base + static_cast<uint32_t>(acc * BN);
        for (int kb = 0; kb < k_blocks; ++kb) {
          if (!mbar_wait(full_bar(stage), phase, abort_word, FT_ERR_TIMEOUT_MMA)) { ok = false; break; }
          tc_fence_after();
          const uint32_t sA = smem_base + stage * Cfg::STAGE_BYTES, sB = sA + Cfg::A_BYTES;
#pragma unroll
          for (int k = 0; k < GG_BK / 16; ++k)
            umma_f16_ss(d_tmem, make_smem_desc_sw128(sA + k * 32, 16, 1024), make_smem_desc_sw128(sB + k * 32, 16, 1024), idesc,
                        (kb > 0 || k > 0) ? 1u : 0u);
          umma_commit(empty_bar(stage));
          if (++stage == STAGES) { stage = 0; phase ^= 1u; }
        }
        if (!ok) break;
        umma_commit(tfull_bar(acc));
        acc ^= 1;
        if (acc == 0) acc_phase ^= 1u;
      }
    }
  } else if (warp >= 4) {
    const int ew = warp & 3, wg = (warp - 4) >> 2;   // TMEM lane quarter; which chunks of the columns
    uint4 u_next[2];                                 // EPI_RGLRU: 16 channels of this lane's row, loaded ahead of the accumulator
    auto fetch_u = [&](const GroupedTile& t, int n, int r) {
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        u_next[q] = make_uint4(0u, 0u, 0u, 0u);
        if (r < t.rows && n + 8 * q < p.N)
          u_next[q] = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.gates.u) +
                                                      (static_cast<long long>(t.row0) + r) * p.gates.ldu + t.group * p.a_col + n + 8 * q);
      }
    };
    int acc = 0;
    uint32_t acc_phase = 0;
    for (int tile = blockIdx.x; tile < num_tiles; tile += gridDim.x) {
      const GroupedTile t = grouped_tile(p, tile, m_items, n_blocks, NW);
      if constexpr (EPI == EPI_RGLRU) fetch_u(t, t.n0 + wg * 16, ew * 32 + lane);
      if (!mbar_wait(tfull_bar(acc), acc_phase, abort_word, FT_ERR_TIMEOUT_EPILOGUE)) break;
      tc_fence_after();
      const uint32_t t_row = tmem_base + (static_cast<uint32_t>(ew * 32) << 16) + static_cast<uint32_t>(acc * BN);
      const int r = ew * 32 + lane;
      const bool row_ok = r < t.rows;
      const long long row = static_cast<long long>(t.row0) + r;
      const bool warp_ok = ew * 32 < t.rows;           // whole warps: the TMEM load is a warp-wide instruction
      float scale = 1.f;
      if constexpr (EPI == EPI_GLU)
        if (p.row_scale && row_ok) scale = p.row_scale[row];
      if constexpr (EPI == EPI_RGLRU) {
        for (int c = wg * 16; warp_ok && c < NW; c += 64) {
          const int n = t.n0 + c;
          if (n >= p.N) break;
          uint32_t za[16], zb[16];
          tmem_ld_32x16(t_row + c, za);
          tmem_ld_32x16(t_row + NW + c, zb);
          tmem_ld_wait();
#pragma unroll
          for (int g = 0; g < 2; ++g) {
            if (!row_ok || n + g * 8 >= p.N) continue;
            const int ch = t.group * p.a_col + n + g * 8;
            float zr[8], zi[8], u8[8], a8[8], x8[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) { zr[e] = __uint_as_float(za[g * 8 + e]); zi[e] = __uint_as_float(zb[g * 8 + e]); }
            unpack8(u_next[g], u8);
            rglru_gates8<__nv_bfloat16>(p.gates, ch, zr, zi, u8, a8, x8);
            if (row < p.gates.n_single) {
              rglru_step8<__nv_bfloat16>(p.gates, row, ch, a8, x8);
            } else {
              store8_sector(p.gates.a + row * p.gates.channels + ch, a8);
              store8_sector(p.gates.x + row * p.gates.channels + ch, x8);
            }
          }
          if (c + 64 < NW) fetch_u(t, n + 64, r);
        }
      } else if (warp_ok) {
#pragma unroll 1
        for (int c = wg * 16; c < NW; c += 32) {
          const int n = t.n0 + c;
          if (n >= p.N) break;
          uint32_t a[16], b[16];
          tmem_ld_32x16(t_row + c, a);
          if constexpr (EPI == EPI_GLU) tmem_ld_32x16(t_row + NW + c, b);
          tmem_ld_wait();
          if (!row_ok) continue;
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            if (n + h * 8 >= p.N) continue;            // N is a multiple of 8
            float f[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) {
              f[e] = __uint_as_float(a[h * 8 + e]);
              if constexpr (EPI == EPI_GLU) f[e] = glu_act(scale * f[e], p.act) * (scale * __uint_as_float(b[h * 8 + e]));
            }
            const long long col = static_cast<long long>(t.group) * p.out_col + n + h * 8;
            if constexpr (EPI == EPI_STORE) {
              if (p.act == GG_RELU2) {
#pragma unroll
                for (int e = 0; e < 8; ++e) { f[e] = fmaxf(f[e], 0.f); f[e] *= f[e]; }
              }
              if (p.gate) {
                float z[8];
                load8(static_cast<const __nv_bfloat16*>(p.gate) + row * p.ldgate + col, z);
#pragma unroll
                for (int e = 0; e < 8; ++e) f[e] *= sigmoid_row(z[e], static_cast<const __nv_bfloat16*>(nullptr));
              }
            }
            store8(static_cast<__nv_bfloat16*>(p.out) + row * p.ldo + col, f);
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(tempty_bar(acc));
      acc ^= 1;
      if (acc == 0) acc_phase ^= 1u;
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

// ----------------------------------------------------------------------------- fp32
// The same problems in fp32 on the CUDA cores: tiles of 64 rows x 32 columns, 256 threads, 4 x 2 sums per part and thread.
constexpr int GF_BM = 64, GF_BN = 32, GF_BK = 16;

template <int EPI>
__global__ void __launch_bounds__(256)
grouped_gemm_f32_kernel(const float* __restrict__ A, const float* __restrict__ W, long long lda, const GroupedParams p) {
  constexpr int PARTS = EPI == EPI_STORE ? 1 : 2;
  __shared__ float sA[GF_BK][GF_BM + 1], sW[PARTS][GF_BK][GF_BN + 1];
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;      // columns 2 tx .., rows 4 ty ..
  const int m_items = grouped_items(p);
  const int n_blocks = (p.N + GF_BN - 1) / GF_BN;
  const int halves = GG_BM / GF_BM;                            // items hold up to GG_BM rows
  for (int tile = blockIdx.x; tile < m_items * halves * n_blocks; tile += gridDim.x) {
    GroupedTile t = grouped_tile(p, tile / halves, m_items, n_blocks, GF_BN);
    const int r0 = (tile % halves) * GF_BM;
    if (r0 >= t.rows) continue;
    float acc[PARTS][4][2];
#pragma unroll
    for (int q = 0; q < PARTS; ++q)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[q][i][0] = acc[q][i][1] = 0.f;
    for (int k0 = 0; k0 < p.K; k0 += GF_BK) {
      __syncthreads();
      for (int i = threadIdx.x; i < GF_BM * GF_BK; i += 256) {
        const int r = i / GF_BK, k = i % GF_BK;
        sA[k][r] = r0 + r < t.rows && k0 + k < p.K ? A[static_cast<long long>(t.row0 + r0 + r) * lda + t.group * p.a_col + k0 + k] : 0.f;
      }
      for (int i = threadIdx.x; i < PARTS * GF_BN * GF_BK; i += 256) {
        const int q = i / (GF_BN * GF_BK), n = i / GF_BK % GF_BN, k = i % GF_BK;
        sW[q][k][n] = t.n0 + n < p.N && k0 + k < p.K
                          ? W[(static_cast<long long>(t.group * p.parts + q) * p.N + t.n0 + n) * p.K + k0 + k] : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int k = 0; k < GF_BK; ++k)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float a = sA[k][ty * 4 + i];
#pragma unroll
          for (int q = 0; q < PARTS; ++q) {
            acc[q][i][0] += a * sW[q][k][tx * 2];
            acc[q][i][1] += a * sW[q][k][tx * 2 + 1];
          }
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = r0 + ty * 4 + i;
      const long long row = static_cast<long long>(t.row0) + r;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int n = t.n0 + tx * 2 + j;
        const bool ok = r < t.rows && n < p.N;
        if constexpr (EPI == EPI_RGLRU) {
          // the gates work on eight neighbouring channels: four threads of a warp exchange theirs
          float zr[8], zi[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const int src = (threadIdx.x & 28) + e / 2;
            const float r0v = __shfl_sync(0xffffffffu, acc[0][i][0], src), r1v = __shfl_sync(0xffffffffu, acc[0][i][1], src);
            const float i0v = __shfl_sync(0xffffffffu, acc[1][i][0], src), i1v = __shfl_sync(0xffffffffu, acc[1][i][1], src);
            zr[e] = e & 1 ? r1v : r0v;
            zi[e] = e & 1 ? i1v : i0v;
          }
          if (j == 0 && (threadIdx.x & 3) == 0 && ok) {
            const int c = t.group * p.a_col + n;
            float u8[8], a8[8], x8[8];
            load8(static_cast<const float*>(p.gates.u) + row * p.gates.ldu + c, u8);
            rglru_gates8<float>(p.gates, c, zr, zi, u8, a8, x8);
            if (row < p.gates.n_single) rglru_step8<float>(p.gates, row, c, a8, x8);
            else {
              store8(p.gates.a + row * p.gates.channels + c, a8);
              store8(p.gates.x + row * p.gates.channels + c, x8);
            }
          }
        } else if (ok) {
          float v = acc[0][i][j];
          if constexpr (EPI == EPI_GLU) {
            const float s = p.row_scale ? p.row_scale[row] : 1.f;
            const float g = s * v;
            v = (p.act == 0 ? g / (1.f + expf(-g)) : glu_act(g, p.act)) * (s * acc[1][i][j]);
          }
          const long long col = static_cast<long long>(t.group) * p.out_col + n;
          if constexpr (EPI == EPI_STORE) {
            if (p.act == GG_RELU2) { v = fmaxf(v, 0.f); v *= v; }
          }
          if constexpr (EPI == EPI_STORE)
            if (p.gate) v *= sigmoid_row(static_cast<const float*>(p.gate)[row * p.ldgate + col], static_cast<const float*>(nullptr));
          static_cast<float*>(p.out)[row * p.ldo + col] = v;
        }
      }
    }
  }
}

// ----------------------------------------------------------------------------- routing
// The experts of a row and their weights from its router logits z.  One warp per row.
//   SCORE_SIGMOID  the `top` largest logits (the lower index of equals), weighted by their sigmoid
//   SCORE_SOFTMAX  scores s = softmax(z) over all outputs; the `top` largest s + correction, weighted by their s, divided by the
//                  sum of these (+ 1e-20) when normalised: the softmax over the chosen logits alone
// A bias per output may join the logits.  One more output behind these may be a gate of the row: its sigmoid is stored.
// With h the logits are computed here, from the row and the router's matrix in fp32 (batches too small for a product of
// their own); else they are read.
constexpr int MR_THREADS = 256;
constexpr int MR_MAX_EXPERTS = 1024;

enum : int { SCORE_SIGMOID = 0, SCORE_SOFTMAX = 1 };

struct RouteRule {
  int outputs, top, score, normalize;   // outputs: router logits of a row
  const float* correction;              // [outputs] or null
  const float* bias;                    // [outputs] or null
  float* gate;                          // [rows] or null: sigmoid of output `outputs`
  __host__ __device__ __forceinline__ int logits() const { return outputs + (gate ? 1 : 0); }
};

// z [rule.logits()] in shared memory is overwritten (softmax scores take a second array of the same size behind it).
__device__ __forceinline__ void choose_experts(float* z, const RouteRule& rule, int lane, long long row, int* index, float* weight) {
  const int n = rule.outputs;
  float* s = z + rule.logits();
  index += row * rule.top;
  weight += row * rule.top;
  if (rule.gate && lane == 0) rule.gate[row] = 1.f / (1.f + expf(-z[n]));
  if (rule.bias) {
    for (int e = lane; e < n; e += 32) z[e] += rule.bias[e];
    __syncwarp();
  }
  if (rule.score == SCORE_SOFTMAX) {
    float m = -INFINITY, sum = 0.f;
    for (int e = lane; e < n; e += 32) m = fmaxf(m, z[e]);
    m = warp_max(m);
    for (int e = lane; e < n; e += 32) {
      s[e] = expf(z[e] - m);
      sum += s[e];
    }
    sum = warp_sum(sum);
    for (int e = lane; e < n; e += 32) {
      s[e] /= sum;
      z[e] = s[e] + (rule.correction ? rule.correction[e] : 0.f);
    }
    __syncwarp();
  }
  float total = 0.f;
  for (int k = 0; k < rule.top; ++k) {
    float best = -INFINITY;
    int at = 0x7fffffff;
    for (int e = lane; e < n; e += 32)
      if (z[e] > best || (z[e] == best && e < at && best > -INFINITY)) { best = z[e]; at = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float b = __shfl_xor_sync(0xffffffffu, best, o);
      const int i = __shfl_xor_sync(0xffffffffu, at, o);
      if (b > best || (b == best && i < at)) { best = b; at = i; }
    }
    if (at >= n) at = k < n ? k : 0;     // logits that are not numbers: still an expert that exists
    const float w = rule.score == SCORE_SOFTMAX ? s[at] : 1.f / (1.f + expf(-best));
    total += w;
    if (lane == 0) {
      index[k] = at;
      weight[k] = w;
      z[at] = -INFINITY;
    }
    __syncwarp();
  }
  if (rule.normalize && lane == 0)
    for (int k = 0; k < rule.top; ++k) weight[k] /= total + 1e-20f;
  __syncwarp();
}

__global__ void __launch_bounds__(MR_THREADS)
moe_choose_kernel(const float* __restrict__ logits, long long ldl, int rows, const RouteRule rule, int* __restrict__ index,
                  float* __restrict__ weight) {
  extern __shared__ float mr_sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = rule.logits();
  float* z = mr_sm + warp * 2 * n;
  for (int row = blockIdx.x * (MR_THREADS / 32) + warp; row < rows; row += gridDim.x * (MR_THREADS / 32)) {
    for (int e = lane; e < n; e += 32) z[e] = logits[row * ldl + e];
    __syncwarp();
    choose_experts(z, rule, lane, row, index, weight);
  }
}

// z[n] = w[n] . h for a row h and n outputs (fp32), in shared or global memory: a warp takes two outputs at a time.
template <typename T>
__device__ __forceinline__ void row_outputs(const T* h, const T* __restrict__ w, int H, int n, float* z) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int e0 = warp * 2; e0 < n; e0 += MR_THREADS / 16) {
    const T* w0 = w + static_cast<long long>(e0) * H;
    const T* w1 = e0 + 1 < n ? w0 + H : w0;
    float s0 = 0.f, s1 = 0.f;
#pragma unroll 4
    for (int i = lane * 8; i < H; i += 256) {
      float a[8], b[8], c[8];
      load8(h + i, a);
      load8(w0 + i, b);
      load8(w1 + i, c);
#pragma unroll
      for (int e = 0; e < 8; ++e) { s0 += a[e] * b[e]; s1 += a[e] * c[e]; }
    }
    s0 = warp_sum(s0);
    s1 = warp_sum(s1);
    if (lane == 0) {
      z[e0] = s0;
      if (e0 + 1 < n) z[e0 + 1] = s1;
    }
  }
}

constexpr int FEW_OUTPUTS = MR_THREADS / 16;       // of a block: two a warp
template <typename T>
__global__ void __launch_bounds__(MR_THREADS)
few_outputs_kernel(const T* __restrict__ h, long long ldh, const T* __restrict__ w, float* __restrict__ z, int rows, int H, int n) {
  const int e0 = blockIdx.y * FEW_OUTPUTS, m = min(FEW_OUTPUTS, n - e0);
  for (int row = blockIdx.x; row < rows; row += gridDim.x)
    row_outputs(h + row * ldh, w + static_cast<long long>(e0) * H, H, m, z + static_cast<long long>(row) * n + e0);
}

// One block per row: the row in registers of all warps in turn, one expert per warp at a time.
template <typename T>
__global__ void __launch_bounds__(MR_THREADS)
moe_route_rows_kernel(const T* __restrict__ h, long long ldh, const T* __restrict__ router, int rows, int H, const RouteRule rule,
                      int* __restrict__ index, float* __restrict__ weight) {
  extern __shared__ float mr_sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int row = blockIdx.x; row < rows; row += gridDim.x) {
    row_outputs(h + row * ldh, router, H, rule.logits(), mr_sm);
    __syncthreads();
    if (warp == 0) choose_experts(mr_sm, rule, lane, row, index, weight);
    __syncthreads();
  }
}

// Sort the (row, choice) pairs by expert.  One block: count, prefix sum, place.  place[i] = sorted position of pair
// i = row * top + k; scale[position] = its weight; items = (expert, first position, rows) with at most GG_BM rows each,
// n_items how many.  Choices of outputs from `experts` on have no rows and place -1.  The order inside an expert is not
// fixed; every row is computed on its own.
__global__ void __launch_bounds__(1024)
moe_build_kernel(const int* __restrict__ index, const float* __restrict__ weight, int pairs, int experts,
                 int* __restrict__ place, float* __restrict__ scale, int* __restrict__ items, int max_items,
                 int* __restrict__ n_items) {
  __shared__ int count[MR_MAX_EXPERTS], base[MR_MAX_EXPERTS], warp_rows[32], warp_items[32];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  count[threadIdx.x] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < pairs; i += 1024)
    if (index[i] < experts) atomicAdd(&count[max(index[i], 0)], 1);
  __syncthreads();
  // exclusive prefix sums of rows and items over the experts (thread = expert)
  const int rows = static_cast<int>(threadIdx.x) < experts ? count[threadIdx.x] : 0;
  const int its = (rows + GG_BM - 1) / GG_BM;
  int pr = rows, pi = its;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int a = __shfl_up_sync(0xffffffffu, pr, o), b = __shfl_up_sync(0xffffffffu, pi, o);
    if (lane >= o) { pr += a; pi += b; }
  }
  if (lane == 31) { warp_rows[warp] = pr; warp_items[warp] = pi; }
  __syncthreads();
  int r0 = pr - rows, i0 = pi - its;
  for (int w = 0; w < warp; ++w) { r0 += warp_rows[w]; i0 += warp_items[w]; }
  base[threadIdx.x] = r0;
  count[threadIdx.x] = 0;
  for (int j = 0; j < its && i0 + j < max_items; ++j) {
    items[3 * (i0 + j)] = threadIdx.x;
    items[3 * (i0 + j) + 1] = r0 + j * GG_BM;
    items[3 * (i0 + j) + 2] = min(GG_BM, rows - j * GG_BM);
  }
  if (threadIdx.x == 1023) *n_items = min(i0 + its, max_items);
  __syncthreads();
  for (int i = threadIdx.x; i < pairs; i += 1024) {
    const int e = max(index[i], 0);
    if (e >= experts) {
      place[i] = -1;
      continue;
    }
    const int at = base[e] + atomicAdd(&count[e], 1);
    place[i] = at;
    scale[at] = weight[i];
  }
}

// out[place[row * top + k]] = h[row]: rows of `units` 16-byte units.
__global__ void moe_permute_kernel(const uint4* __restrict__ h, long long ldh16, const int* __restrict__ place, uint4* __restrict__ out,
                                   int rows, int top, int units) {
  for (int row = blockIdx.x; row < rows; row += gridDim.x)
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < units; i += gridDim.y * blockDim.x) {
      const uint4 v = h[row * ldh16 + i];
      for (int k = 0; k < top; ++k) {
        const int at = place[row * top + k];
        if (at >= 0 && at < rows * top) out[static_cast<long long>(at) * units + i] = v;
      }
    }
}

template <int BN, int EPI>
static int launch_grouped(const CUtensorMap& ta, const CUtensorMap& tb, const GroupedParams& p, long long tiles, int device,
                          cudaStream_t stream) {
  using Cfg = GgCfg<BN, EPI>;
  auto kern = grouped_gemm_kernel<BN, EPI>;
  static bool attr_set[64] = {false};
  if (!attr_set[device]) {
    FT_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM_BYTES));
    attr_set[device] = true;
  }
  const int sms = sm_count(device);
  kern<<<tiles < sms ? static_cast<int>(tiles) : sms, Cfg::THREADS, Cfg::SMEM_BYTES, stream>>>(ta, tb, p);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// Shared host side: shapes, tensor maps, tile width.  lda in elements; total_rows: rows of A.
template <int EPI>
static int run_grouped(const void* A, long long lda, int total_rows, const void* W, GroupedParams& p, int f32, int bn, int device,
                       cudaStream_t stream) {
  p.parts = EPI == EPI_STORE ? 1 : 2;
  const int item_bound = p.items ? p.max_items : p.groups * ((p.rows + GG_BM - 1) / GG_BM);
  if (item_bound <= 0 || total_rows <= 0) return FT_E_OK;
  if (f32) {
    const long long tiles = static_cast<long long>(item_bound) * (GG_BM / GF_BM) * ((p.N + GF_BN - 1) / GF_BN);
    const int cap = sm_count(device) * 8;
    grouped_gemm_f32_kernel<EPI><<<tiles < cap ? static_cast<int>(tiles) : cap, 256, 0, stream>>>(
        static_cast<const float*>(A), static_cast<const float*>(W), lda, p);
    FT_CUDA_CHECK(cudaGetLastError());
    count_launch();
    return FT_E_OK;
  }
  p.status = device_status_word(device);
  auto tiles_at = [&](int width) { return static_cast<long long>(item_bound) * ((p.N + width / p.parts - 1) / (width / p.parts)); };
  if (bn == 0) {
    bn = 256;
    while (bn > 64 && (tiles_at(bn) < sm_count(device) || p.N <= bn / p.parts / 2)) bn >>= 1;
  }
  FT_REQUIRE(bn == 64 || bn == 128 || bn == 256, "grouped gemm: tile width %d", bn);
  CUtensorMap ta, tb;
  const uint64_t inner = p.a_col ? static_cast<uint64_t>(p.groups - 1) * p.a_col + p.K : p.K;
  int rc = make_tmap_2d(&ta, A, 2, inner, total_rows, static_cast<uint64_t>(lda) * 2, GG_BK, p.a_rows, 3);
  if (rc) return rc;
  rc = make_tmap_2d(&tb, W, 2, p.K, static_cast<uint64_t>(p.groups) * p.parts * p.N, static_cast<uint64_t>(p.K) * 2, GG_BK, bn / 2, 3);
  if (rc) return rc;
  if (bn == 256) return launch_grouped<256, EPI>(ta, tb, p, tiles_at(256), device, stream);
  if (bn == 128) return launch_grouped<128, EPI>(ta, tb, p, tiles_at(128), device, stream);
  return launch_grouped<64, EPI>(ta, tb, p, tiles_at(64), device, stream);
}

static bool gg_aligned(std::initializer_list<const void*> ps) {
  uintptr_t v = 0;
  for (const void* p : ps) v |= reinterpret_cast<uintptr_t>(p);
  return (v & 15) == 0;
}

}  // namespace ft

using namespace ft;

// z [rows, n] = h [rows, H] w^T, fp32 results for a few outputs n of few rows (more of either: a product of their own).  h and w bf16,
// or fp32 with f32; H a multiple of 8.
FT_API int ft_few_outputs(const void* h, long long ldh, const void* w, float* z, int rows, int H, int n, int f32, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(h && w && z && H > 0 && H % 8 == 0 && ldh % 8 == 0 && n > 0 && gg_aligned({h, w}), "ft_few_outputs: H=%d and strides must be multiples of 8", H);
  if (rows <= 0) return FT_E_OK;
  const int cap = sm_count(device) * 8;
  const dim3 grid(rows < cap ? rows : cap, (n + FEW_OUTPUTS - 1) / FEW_OUTPUTS);
  if (f32) few_outputs_kernel<float><<<grid, MR_THREADS, 0, stream>>>(static_cast<const float*>(h), ldh, static_cast<const float*>(w), z, rows, H, n);
  else few_outputs_kernel<__nv_bfloat16><<<grid, MR_THREADS, 0, stream>>>(static_cast<const __nv_bfloat16*>(h), ldh, static_cast<const __nv_bfloat16*>(w), z, rows, H, n);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// Work items that ft_moe_route can list for `pairs` (row, choice) pairs over `experts`.
FT_API int ft_moe_max_items(int pairs, int experts) { return (pairs < experts ? pairs : experts) + pairs / GG_BM; }

// Routing of `rows` rows (see RouteRule): the choices of every row and their weights, rows sorted by expert.  The router has
// outputs >= experts logits; choices from `experts` on have no matrices: place -1.  logits: fp32 [rows, ldl] or null (then
// computed from h and router [outputs, H], the type of h).  bias fp32 [outputs] or null joins the logits.  gate fp32 [rows] or null: the
// router has one more output, whose sigmoid this receives.  Outputs: index int32 [rows, top], weight fp32 [rows, top], place
// int32 [rows, top] (sorted position), scale fp32 [rows * top] (by position), items int32 [max_items, 3] and n_items for
// ft_grouped_gemm, sorted [rows * top, H] (the rows of h).  h: bf16, or fp32 with f32; H a multiple of 8; outputs <= 1024.
FT_API int ft_moe_route(const void* h, long long ldh, const void* router, const float* logits, long long ldl, int rows, int H,
                        int experts, int outputs, int top, int score, const float* correction, const float* bias, int normalize,
                        float* gate, int f32, int* index, float* weight, int* place, float* scale, int* items, int max_items, int* n_items, void* sorted, int device,
                        cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(h && (router || logits) && index && weight && place && scale && items && n_items && sorted, "ft_moe_route: null pointer");
  FT_REQUIRE(experts >= 1 && outputs >= experts && outputs <= MR_MAX_EXPERTS && top >= 1 && top <= outputs, "ft_moe_route: %d of %d outputs, %d experts", top, outputs, experts);
  FT_REQUIRE(outputs + (gate ? 1 : 0) <= MR_MAX_EXPERTS, "ft_moe_route: %d outputs and a gate", outputs);
  FT_REQUIRE(score == SCORE_SOFTMAX || (score == SCORE_SIGMOID && !correction), "ft_moe_route: score %d", score);
  FT_REQUIRE(H > 0 && H % 8 == 0 && ldh % 8 == 0 && gg_aligned({h, router, sorted}), "ft_moe_route: H=%d and strides must be multiples of 8", H);
  FT_REQUIRE(static_cast<long long>(rows) * top < (1ll << 31) && max_items >= ft_moe_max_items(rows * top, experts), "ft_moe_route: %d items are too few", max_items);
  if (rows <= 0) return FT_E_OK;
  const int sms = sm_count(device);
  const RouteRule rule = {outputs, top, score, normalize, correction, bias, gate};
  if (logits) {
    const size_t smem = static_cast<size_t>(MR_THREADS / 32) * 2 * rule.logits() * sizeof(float);
    const int need = (rows + MR_THREADS / 32 - 1) / (MR_THREADS / 32), cap = sms * 8;
    FT_CUDA_CHECK(cudaFuncSetAttribute(moe_choose_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    moe_choose_kernel<<<need < cap ? need : cap, MR_THREADS, smem, stream>>>(logits, ldl, rows, rule, index, weight);
  } else {
    const int cap = sms * 8;
    const size_t smem = static_cast<size_t>(rule.logits()) * 2 * sizeof(float);
    if (f32)
      moe_route_rows_kernel<float><<<rows < cap ? rows : cap, MR_THREADS, smem, stream>>>(
          static_cast<const float*>(h), ldh, static_cast<const float*>(router), rows, H, rule, index, weight);
    else
      moe_route_rows_kernel<__nv_bfloat16><<<rows < cap ? rows : cap, MR_THREADS, smem, stream>>>(
          static_cast<const __nv_bfloat16*>(h), ldh, static_cast<const __nv_bfloat16*>(router), rows, H, rule, index, weight);
  }
  FT_CUDA_CHECK(cudaGetLastError());
  moe_build_kernel<<<1, 1024, 0, stream>>>(index, weight, rows * top, experts, place, scale, items, max_items, n_items);
  FT_CUDA_CHECK(cudaGetLastError());
  const int unit = f32 ? 4 : 8, units = H / unit;
  int parts = (units + 255) / 256;
  if (parts > sms * 8 / rows) parts = sms * 8 / rows > 1 ? sms * 8 / rows : 1;
  const int cap = sms * 16;
  moe_permute_kernel<<<dim3(rows < cap ? rows : cap, parts), units < 256 ? (units + 31) / 32 * 32 : 256, 0, stream>>>(
      static_cast<const uint4*>(h), ldh / unit, place, static_cast<uint4*>(sorted), rows, top, units);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch(3);
  return FT_E_OK;
}

// out = epilogue(A W^T) over segments of rows: A [total_rows, K], W [groups, parts, N, K], items / n_items as
// ft_moe_route writes them (at most max_items).  glu 0: one part, out = the sum, or with act 3 the square of its relu; glu 1: two parts (gate, up), out =
// act(r gate) * (r up) with r = row_scale (null: 1), act 0 silu / 1 relu / 2 gelu (tanh form).  seg_rows: an upper
// bound of the rows of a segment (0: none known).  All bf16, or fp32 with f32.  N and K multiples of 8.
FT_API int ft_grouped_gemm(const void* A, long long lda, int total_rows, const void* W, const int* items, const int* n_items,
                           int max_items, int groups, int N, int K, int glu, const float* row_scale, int act, void* out,
                           long long ldo, int seg_rows, int f32, int bn, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(A && W && items && n_items && out, "ft_grouped_gemm: null pointer");
  FT_REQUIRE(groups > 0 && N > 0 && K > 0 && ((N | K) & 7) == 0 && lda % 8 == 0 && ldo % 8 == 0 && lda >= K && ldo >= N,
             "ft_grouped_gemm: N=%d, K=%d and strides must be multiples of 8", N, K);
  FT_REQUIRE(gg_aligned({A, W, out}), "ft_grouped_gemm: pointers must be 16-byte aligned");
  FT_REQUIRE((glu ? act >= 0 && act <= 2 : act == 0 || act == GG_RELU2) && static_cast<long long>(groups) * 2 * N < (1ll << 31), "ft_grouped_gemm: bad argument");
  GroupedParams p = {};
  p.items = items; p.n_items_dev = n_items; p.max_items = max_items; p.groups = groups;
  p.a_rows = GG_BM;
  if (seg_rows > 0)
    while (p.a_rows > 16 && p.a_rows / 2 >= seg_rows) p.a_rows >>= 1;
  p.N = N; p.K = K; p.out = out; p.ldo = ldo; p.row_scale = row_scale; p.act = act;
  return glu ? run_grouped<EPI_GLU>(A, lda, total_rows, W, p, f32, bn, device, stream)
             : run_grouped<EPI_STORE>(A, lda, total_rows, W, p, f32, bn, device, stream);
}

// The same product over blocks of columns: group g multiplies columns g * a_col .. g * a_col + K - 1 of every row of A [rows, lda]
// by W [groups, parts, N, K] into columns g * out_col .. of out.  glu as in ft_grouped_gemm; gate (glu 0; [rows, ldgate], null: none):
// every result is multiplied by the sigmoid of the gate at its row and column.  Sizes and strides multiples of 8.
FT_API int ft_block_linear(const void* A, long long lda, int rows, const void* W, int groups, int a_col, int N, int K, int glu, int act,
                           void* out, long long ldo, int out_col, const void* gate, long long ldgate, int f32, int bn, int device,
                           cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(A && W && out && !(gate && glu), "ft_block_linear: null pointer, or a gate with glu");
  FT_REQUIRE(groups > 0 && N > 0 && K > 0 && ((N | K | a_col | out_col) & 7) == 0 && ((lda | ldo | ldgate) & 7) == 0 && K <= a_col &&
                 (out_col >= N || groups == 1) && lda >= static_cast<long long>(groups - 1) * a_col + K &&
                 ldo >= static_cast<long long>(groups - 1) * out_col + N && (!gate || ldgate >= static_cast<long long>(groups - 1) * out_col + N),
             "ft_block_linear: %d blocks of N=%d, K=%d", groups, N, K);
  FT_REQUIRE(gg_aligned({A, W, out, gate}), "ft_block_linear: pointers must be 16-byte aligned");
  FT_REQUIRE(act >= 0 && act <= 2 && static_cast<long long>(groups) * 2 * N < (1ll << 31), "ft_block_linear: bad argument");
  if (rows <= 0) return FT_E_OK;
  GroupedParams p = {};
  p.rows = rows; p.groups = groups; p.a_col = a_col; p.a_rows = GG_BM; p.N = N; p.K = K;
  while (p.a_rows > 16 && p.a_rows / 2 >= rows) p.a_rows >>= 1;
  p.out = out; p.ldo = ldo; p.out_col = out_col; p.act = act; p.gate = gate; p.ldgate = ldgate;
  return glu ? run_grouped<EPI_GLU>(A, lda, rows, W, p, f32, bn, device, stream)
             : run_grouped<EPI_STORE>(A, lda, rows, W, p, f32, bn, device, stream);
}

// Gates of a real-gated linear recurrence for all rows, from u [rows, ldu] (blocks * n channels) and W [blocks, 2, n, n]
// (r and i matrices): decay a and input term x, fp32 [rows, channels], for rows n_single ..; rows before that are single
// tokens of their sequences and finish here: state [slots, channels] takes its step, out [rows, ldo] = state * gelu(y).
// r_bias, i_bias, decay: fp32 [channels].  u, W, y, out bf16, or fp32 with f32.  n a multiple of 8.
FT_API int ft_rglru_gates(const void* u, long long ldu, const void* W, const float* r_bias, const float* i_bias, const float* decay,
                          int rows, int blocks, int n, float* a, float* x, int n_single, const int* pos, const int* slots,
                          float* state, const void* y, long long ldy, void* out, long long ldo, int f32, int bn, int device,
                          cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(u && W && r_bias && i_bias && decay && a && x && pos && slots && state && y && out, "ft_rglru_gates: null pointer");
  FT_REQUIRE(blocks > 0 && n > 0 && n % 8 == 0 && ((ldu | ldy | ldo) & 7) == 0 && ldu >= static_cast<long long>(blocks) * n &&
                 ldy >= static_cast<long long>(blocks) * n && ldo >= static_cast<long long>(blocks) * n,
             "ft_rglru_gates: block size %d and strides must be multiples of 8", n);
  FT_REQUIRE(gg_aligned({u, W, r_bias, i_bias, decay, state, y, out}) &&
                 ((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(x)) & 31) == 0,
             "ft_rglru_gates: pointers must be 16-byte aligned, a and x 32-byte");
  FT_REQUIRE(n_single >= 0 && n_single <= rows, "ft_rglru_gates: %d single rows of %d", n_single, rows);
  if (rows <= 0) return FT_E_OK;
  GroupedParams p = {};
  p.rows = rows; p.groups = blocks; p.a_col = n; p.a_rows = GG_BM; p.N = n; p.K = n;
  while (p.a_rows > 16 && p.a_rows / 2 >= rows) p.a_rows >>= 1;
  RglruGateParams& g = p.gates;
  g.u = u; g.r_bias = r_bias; g.i_bias = i_bias; g.decay = decay; g.a = a; g.x = x; g.ldu = ldu;
  g.channels = blocks * n; g.n_single = n_single; g.pos = pos; g.slots = slots; g.state = state;
  g.y = y; g.out = out; g.ldy = ldy; g.ldo = ldo;
  return run_grouped<EPI_RGLRU>(u, ldu, rows, W, p, f32, bn, device, stream);
}
