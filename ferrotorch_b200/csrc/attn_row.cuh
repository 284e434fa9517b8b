// Arithmetic that attention kernels share: one row of a 128 x 128 score tile kept in registers (attn_fwd.cu,
// paged_prefill.cu); windows, sinks and output gates (paged_attn.cu, paged_prefill.cu).
#pragma once
#include "ft_ptx.cuh"

namespace ft {

constexpr int ATT_BM = 128;   // query rows of a tile
constexpr int ATT_BN = 128;   // keys of a tile
// A row keeps its reference maximum until the true maximum has moved by more than this many powers of two.
constexpr float ATT2_RESCALE_THRESHOLD = 8.f;

// p = 2^(s * scale + neg_m) for one row of 128 scores held as packed pairs; writes the bf16 pairs
// and returns the row sum (four independent partial sums of pairs).  Moving a share of the
// exponentials from the special-function unit to a polynomial on the FMA pipe was measured at
// 0 / 25 / 37 / 50 / 62 %: 908 / 904 / 902 / 880 / 811 TFLOP/s at B4 S4096 H32/8 D128, so all of
// them stay on ex2.approx.
__device__ __forceinline__ float att2_exp_row(const f32x2 (&sp)[ATT_BN / 2], float scale, float neg_m,
                                              uint32_t (&pk)[ATT_BN / 2]) {
  const f32x2 sc2 = f2_pack(scale, scale), nm2 = f2_pack(neg_m, neg_m);
  f32x2 acc[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) acc[k] = f2_pack(0.f, 0.f);
#pragma unroll
  for (int i = 0; i < ATT_BN / 2; ++i) {
    float x0, x1;
    f2_unpack(f2_fma(sp[i], sc2, nm2), x0, x1);
    const float e0 = fast_exp2(x0), e1 = fast_exp2(x1);
    acc[i & 3] = f2_add(acc[i & 3], f2_pack(e0, e1));
    pk[i] = pack_bf16x2(e0, e1);
  }
  float a, b, c, d;
  f2_unpack(f2_add(acc[0], acc[1]), a, b);
  f2_unpack(f2_add(acc[2], acc[3]), c, d);
  return (a + b) + (c + d);
}

// The row (128 fp32 scores starting at TMEM column s_addr) as 64 packed pairs.
__device__ __forceinline__ void att2_load_row(uint32_t s_addr, f32x2 (&sp)[ATT_BN / 2]) {
  uint32_t t0[32], t1[32], t2[32], t3[32];
  tmem_ld_32x32(s_addr, t0);
  tmem_ld_32x32(s_addr + 32, t1);
  tmem_ld_32x32(s_addr + 64, t2);
  tmem_ld_32x32(s_addr + 96, t3);
  tmem_ld_wait();
#pragma unroll
  for (int i = 0; i < 16; ++i) {
    sp[i] = f2_pack(__uint_as_float(t0[2 * i]), __uint_as_float(t0[2 * i + 1]));
    sp[16 + i] = f2_pack(__uint_as_float(t1[2 * i]), __uint_as_float(t1[2 * i + 1]));
    sp[32 + i] = f2_pack(__uint_as_float(t2[2 * i]), __uint_as_float(t2[2 * i + 1]));
    sp[48 + i] = f2_pack(__uint_as_float(t3[2 * i]), __uint_as_float(t3[2 * i + 1]));
  }
}

// Keys past the last visible one (kv0 + c > limit) get -inf.
__device__ __forceinline__ void att2_mask_row(f32x2 (&sp)[ATT_BN / 2], int kv0, int limit) {
#pragma unroll
  for (int i = 0; i < ATT_BN / 2; ++i) {
    float a, b;
    f2_unpack(sp[i], a, b);
    if (kv0 + 2 * i > limit) a = -INFINITY;
    if (kv0 + 2 * i + 1 > limit) b = -INFINITY;
    sp[i] = f2_pack(a, b);
  }
}

// Keys ahead of the first visible one (kv0 + c < first) get -inf.
__device__ __forceinline__ void att2_mask_ahead(f32x2 (&sp)[ATT_BN / 2], int kv0, int first) {
#pragma unroll
  for (int i = 0; i < ATT_BN / 2; ++i) {
    float a, b;
    f2_unpack(sp[i], a, b);
    if (kv0 + 2 * i < first) a = -INFINITY;
    if (kv0 + 2 * i + 1 < first) b = -INFINITY;
    sp[i] = f2_pack(a, b);
  }
}

__device__ __forceinline__ float att2_row_max(const f32x2 (&sp)[ATT_BN / 2]) {
  float m0 = -INFINITY, m1 = -INFINITY, m2 = -INFINITY, m3 = -INFINITY;   // four independent chains
#pragma unroll
  for (int i = 0; i < ATT_BN / 2; i += 4) {
    float a, b;
    f2_unpack(sp[i], a, b);
    m0 = max3(m0, a, b);
    f2_unpack(sp[i + 1], a, b);
    m1 = max3(m1, a, b);
    f2_unpack(sp[i + 2], a, b);
    m2 = max3(m2, a, b);
    f2_unpack(sp[i + 3], a, b);
    m3 = max3(m3, a, b);
  }
  return fmaxf(max3(m0, m1, m2), m3);
}

// ---------------------------------------------------------------- visible keys, distance bias, sink, output gate
// A query at position len - 1 sees keys first_visible .. len - 1: with a window the last so many, with chunks (counted from
// position 0) those of its own chunk; 0: no such limit.
struct KeyRange {
  int window, chunk;
  __device__ __forceinline__ int first_visible(int len) const {
    const int lo = window > 0 ? max(0, len - window) : 0;
    return chunk > 0 ? max(lo, max(len - 1, 0) / chunk * chunk) : lo;
  }
};

// Means of keys and values over blocks of `pool` consecutive positions (counted from 0), seen once a block lies wholly ahead of
// the window.  Block b lies with the page that holds its last position: [num_blocks, per_page, Hkv, head size].
struct PooledKeys {
  const void* k;
  const void* v;
  int pool, per_page;      // pool 0: none
  // Blocks that a query sees whose first visible key is `first`.
  __device__ __forceinline__ int count(int first) const { return pool > 0 ? first / pool : 0; }
  // Row of block b on the [num_blocks * per_page] axis; bt: the sequence's pages.
  __device__ __forceinline__ long long row(int b, const int* bt, int block_size, int max_blocks, int num_blocks) const {
    const int page = min((b * pool + pool - 1) / block_size, max_blocks - 1);
    const int at = min(max(b - page * block_size / pool, 0), per_page - 1);
    return static_cast<long long>(min(max(__ldg(bt + page), 0), num_blocks - 1)) * per_page + at;
  }
};
static inline PooledKeys pooled_keys(const void* k, const void* v, int pool, int block_size) {
  return PooledKeys{k, v, pool, pool > 0 ? (block_size - 1) / pool + 1 : 0};
}
constexpr float ATT_LOG2E = 1.4426950408889634f;

// A head's sink joins the softmax: exp(sink) in the denominator, no key, no value, no scale.  m, l and acc are the
// running maximum (in powers of two), the sum and an output element relative to that maximum.
__device__ __forceinline__ void sink_join(const float* sink, int head, float& m, float& l, float& acc) {
  if (!sink) return;
  const float s2 = sink[head] * 1.4426950408889634f;
  const float mm = fmaxf(m, s2);
  const float sc = m == -INFINITY ? 0.f : exp2f(m - mm);
  l = l * sc + exp2f(s2 - mm);
  acc *= sc;
  m = mm;
}

// Output gate: element d of head h of a row is multiplied by sigmoid(g[row * ld + h * head + d * elem]).
struct HeadGate {
  const void* g;       // null: no gate
  long long ld;
  int head, elem;      // strides; elem 0: one number per head
  __device__ __forceinline__ long long at(int row, int h, int d) const {
    return row * ld + static_cast<long long>(h) * head + static_cast<long long>(d) * elem;
  }
};
__device__ __forceinline__ float gate_value(float z) { return 1.f / (1.f + expf(-z)); }
// The same ahead of a bf16 store: approximate exponential and division (an epilogue applies it to every output element).
__device__ __forceinline__ float gate_value_bf16(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }
__device__ __forceinline__ float head_gate_bf16(const HeadGate& gt, int row, int head, int d) {
  if (!gt.g) return 1.f;
  return gate_value_bf16(__bfloat162float(static_cast<const __nv_bfloat16*>(gt.g)[gt.at(row, head, d)]));
}

}  // namespace ft
