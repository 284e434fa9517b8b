// Row kernels of decoders with an fp32 residual stream:
//
//   ft_rms_rows        RMS norm of residual rows, optionally gathering the rows first (the embedding,
//                      or the rows whose logits are wanted) and optionally adding pending terms to the
//                      residual (the outputs of a token's experts), all in one pass over the row.
//   ft_sum_norm_rows   norm after the sum: a factor times the residual row plus a sublayer's terms times their gate,
//                      RMS-normed back into the residual and into the next sublayer's input, in one pass.
//   ft_part_norm       RMS norm of equal runs of a row on their own, in place.
//   ft_poly_norm       sum of a row's first three powers, each over its own root mean square.
//   ft_qkv_head_finish everything between a packed projection [ q | k | v | .. ] and its attention:
//                      per-head RMS norm of q and k, rotation of the first 2 * half elements of a head
//                      by a cos / sin table, k and v into their cache pages.
//
// Rows are bf16 or fp32, arithmetic is fp32.
#include <initializer_list>

#include "recurrent.cuh"
#include "row_vec.cuh"

namespace ft {

constexpr int ROW_THREADS = 256;
constexpr int ROW_WARPS = ROW_THREADS / 32;
constexpr int ROW_KEEP = 2;   // vectors of eight elements a thread keeps in registers (rows up to 4096 wide)

struct RmsRowsParams {
  const void* x;            // [n_src, ldx]
  const long long* ids;     // row i reads x[ids[i]] (null: x[i])
  float* x_out;             // fp32 [rows, ldo]: the row with its terms (may be x itself); null: not written
  const void* terms;        // [.., ldt]: row i gains terms[where[source row * n_terms + j]], j < n_terms
  const int* where;
  const float* w;
  void* y;                  // [rows, ldy]
  long long ldx, ldo, ldt, ldy;
  int rows, n_src, H, count, n_terms, term_rows;
  float eps, offset;
};

// y = x / sqrt(sum(x^2) / count + eps) * (offset + w).  One block per row.
template <typename TI, typename TO>
__global__ void __launch_bounds__(ROW_THREADS)
rms_rows_kernel(const RmsRowsParams p) {
  __shared__ float red[ROW_WARPS];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x) {
    long long src = row;
    if (p.ids) {
      src = p.ids[row];
      if (src < 0 || src >= p.n_src) src = 0;    // host validates; never read out of range
    }
    const TI* xr = static_cast<const TI*>(p.x) + src * p.ldx;
    float* xo = p.x_out ? p.x_out + static_cast<long long>(row) * p.ldo : nullptr;
    TO* yr = static_cast<TO*>(p.y) + static_cast<long long>(row) * p.ldy;
    auto fetch = [&](int i, float (&f)[8]) {
      load8(xr + i, f);
      for (int j = 0; j < p.n_terms; ++j) {
        const int t = p.where[src * p.n_terms + j];
        if (t < 0 || t >= p.term_rows) continue;
        float g[8];
        load8(static_cast<const TO*>(p.terms) + static_cast<long long>(t) * p.ldt + i, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] += g[e];
      }
    };
    float kept[ROW_KEEP][8];
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < ROW_KEEP; ++k) {
      const int i = (k * ROW_THREADS + threadIdx.x) * 8;
      if (i < p.H) {
        fetch(i, kept[k]);
        if (xo) store8(xo + i, kept[k]);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum += kept[k][e] * kept[k][e];
      }
    }
    const int rest = ROW_KEEP * ROW_THREADS * 8 + threadIdx.x * 8;
    // wider rows: the tail is summed here and fetched once more below (a thread owns the same columns in both
    // passes, so with x_out == x it must not add the terms again)
    for (int i = rest; i < p.H; i += ROW_THREADS * 8) {
      float f[8];
      fetch(i, f);
      if (xo) store8(xo + i, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) sum += f[e] * f[e];
    }
    sum = warp_sum(sum);
    __syncthreads();                       // the previous row's sums have been read
    if (lane == 0) red[warp] = sum;
    __syncthreads();
    sum = 0.f;
#pragma unroll
    for (int w = 0; w < ROW_WARPS; ++w) sum += red[w];
    const float r = 1.f / sqrtf(sum / static_cast<float>(p.count) + p.eps);
#pragma unroll
    for (int k = 0; k < ROW_KEEP; ++k) {
      const int i = (k * ROW_THREADS + threadIdx.x) * 8;
      if (i < p.H) {
        float w[8];
        load8(p.w + i, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) w[e] = kept[k][e] * r * (p.offset + w[e]);
        store8(yr + i, w);
      }
    }
    for (int i = rest; i < p.H; i += ROW_THREADS * 8) {
      float f[8], w[8];
      if (xo) load8(static_cast<const float*>(xo) + i, f); else fetch(i, f);
      load8(p.w + i, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) w[e] = f[e] * r * (p.offset + w[e]);
      store8(yr + i, w);
    }
  }
}

// ---------------------------------------------------------------- norm after the sum
struct SumNormParams {
  const void* x;            // [n_src, ldx]
  const long long* ids;     // token i has x[ids[i]] (null: x[i])
  const long long* rows;    // row i is token rows[i] (null: token i)
  const void* dense;        // [tokens, ldd] or null, times dense_weight[token] (null: 1)
  const float* dense_weight;
  const void* terms;        // [term_rows, ldt]: token i gains weight[i, j] (null: 1) times terms[where[i, j]], j < n_terms
  const int* where;
  const float* weight;
  const void* gate;         // [tokens, ldg] or null: the terms' sum is multiplied by its sigmoid
  const float* w;           // [H]
  const float* w2;          // [H]: of a second norm ahead of h; null: none
  float* x_out;             // fp32 [rows, ldo] or null; may be x when ids and rows are null
  void* h;                  // [rows, ldh] or null
  long long ldx, ldd, ldt, ldg, ldo, ldh;
  int n_rows, tokens, n_src, H, count, n_terms, term_rows;
  float alpha, eps;
};

__device__ __forceinline__ float block_total(float v, float* red) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  v = warp_sum(v);
  __syncthreads();                         // the previous total has been read
  if (lane == 0) red[warp] = v;
  __syncthreads();
  v = 0.f;
#pragma unroll
  for (int w = 0; w < ROW_WARPS; ++w) v += red[w];
  return v;
}

// One block per row.
template <typename TI, typename TO>
__global__ void __launch_bounds__(ROW_THREADS, 4)
sum_norm_rows_kernel(const SumNormParams p) {
  __shared__ float red[ROW_WARPS];
  for (int row = blockIdx.x; row < p.n_rows; row += gridDim.x) {
    long long token = row;
    if (p.rows) {
      token = p.rows[row];
      if (token < 0 || token >= p.tokens) token = 0;    // host validates; never read out of range
    }
    long long src = token;
    if (p.ids) {
      src = p.ids[token];
      if (src < 0 || src >= p.n_src) src = 0;
    }
    const TI* xr = static_cast<const TI*>(p.x) + src * p.ldx;
    const TO* dr = p.dense ? static_cast<const TO*>(p.dense) + token * p.ldd : nullptr;
    const TO* gr = p.gate ? static_cast<const TO*>(p.gate) + token * p.ldg : nullptr;
    const float dw = p.dense_weight ? p.dense_weight[token] : 1.f;
    const int* where = p.where + token * p.n_terms;
    const float* weight = p.weight ? p.weight + token * p.n_terms : nullptr;
    float* xo = p.x_out ? p.x_out + static_cast<long long>(row) * p.ldo : nullptr;
    TO* hr = p.h ? static_cast<TO*>(p.h) + static_cast<long long>(row) * p.ldh : nullptr;
    auto fetch = [&](int i, float (&f)[8]) {
      float y[8], g[8];
      load8(xr + i, f);
      if (gr) load8(gr + i, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = 0.f;
      if (dr) {
        load8(dr + i, y);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] *= dw;
      }
      for (int j = 0; j < p.n_terms; ++j) {
        const int t = where[j];
        const float wt = weight ? weight[j] : 1.f;
        if (t < 0 || t >= p.term_rows) continue;
        float z[8];
        load8(static_cast<const TO*>(p.terms) + static_cast<long long>(t) * p.ldt + i, z);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] += wt * z[e];
      }
      if (gr) {
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] *= sigmoid_row(g[e], static_cast<const TO*>(nullptr));
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = p.alpha * f[e] + y[e];
    };
    float kept[ROW_KEEP][8];
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < ROW_KEEP; ++k) {
      const int i = (k * ROW_THREADS + threadIdx.x) * 8;
      if (i < p.H) {
        fetch(i, kept[k]);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum += kept[k][e] * kept[k][e];
      }
    }
    // wider rows: the tail's sum waits in x_out where there is one (a thread owns the same columns in every pass) and is formed
    // anew where not
    const int rest = ROW_KEEP * ROW_THREADS * 8 + threadIdx.x * 8;
    for (int i = rest; i < p.H; i += ROW_THREADS * 8) {
      float f[8];
      fetch(i, f);
      if (xo) store8(xo + i, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) sum += f[e] * f[e];
    }
    const float r = 1.f / sqrtf(block_total(sum, red) / static_cast<float>(p.count) + p.eps);
    auto normed = [&](int i, const float (&f)[8], float (&o)[8]) {
      float w[8];
      load8(p.w + i, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) o[e] = f[e] * r * w[e];
    };
    float r2 = 1.f;
    if (p.w2) {
      sum = 0.f;
#pragma unroll
      for (int k = 0; k < ROW_KEEP; ++k) {
        const int i = (k * ROW_THREADS + threadIdx.x) * 8;
        if (i < p.H) {
          float o[8];
          normed(i, kept[k], o);
#pragma unroll
          for (int e = 0; e < 8; ++e) sum += o[e] * o[e];
        }
      }
      for (int i = rest; i < p.H; i += ROW_THREADS * 8) {
        float f[8], o[8];
        if (xo) load8(static_cast<const float*>(xo) + i, f); else fetch(i, f);
        normed(i, f, o);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum += o[e] * o[e];
      }
      r2 = 1.f / sqrtf(block_total(sum, red) / static_cast<float>(p.count) + p.eps);
    }
    auto store = [&](int i, const float (&f)[8]) {
      float o[8];
      normed(i, f, o);
      if (xo) store8(xo + i, o);
      if (!hr) return;
      if (p.w2) {
        float w[8];
        load8(p.w2 + i, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] *= r2 * w[e];
      }
      store8(hr + i, o);
    };
#pragma unroll
    for (int k = 0; k < ROW_KEEP; ++k) {
      const int i = (k * ROW_THREADS + threadIdx.x) * 8;
      if (i < p.H) store(i, kept[k]);
    }
    for (int i = rest; i < p.H; i += ROW_THREADS * 8) {
      float f[8];
      if (xo) load8(static_cast<const float*>(xo) + i, f); else fetch(i, f);
      store(i, f);
    }
  }
}

// ---------------------------------------------------------------- norms inside sublayers
constexpr int PN_KEEP = 4;      // vectors of eight elements a thread keeps in registers

// `parts` runs of n elements per row, contiguous and whole vectors; GT threads take one run.
template <typename T, int GT>
__global__ void __launch_bounds__(ROW_THREADS)
part_norm_kernel(T* __restrict__ y, long long ld, const float* __restrict__ w, int rows, int parts, int n, float eps) {
  __shared__ float red[ROW_WARPS];
  const int t = threadIdx.x % GT;
  const long long tasks = static_cast<long long>(rows) * parts;
  for (long long task = static_cast<long long>(blockIdx.x) * (ROW_THREADS / GT) + threadIdx.x / GT; task < tasks;
       task += static_cast<long long>(gridDim.x) * (ROW_THREADS / GT)) {
    const long long row = task / parts;
    const int part = static_cast<int>(task - row * parts);
    T* at = y + row * ld + static_cast<long long>(part) * n;
    const float* wp = w + static_cast<long long>(part) * n;
    float kept[PN_KEEP][8];
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < PN_KEEP; ++k) {
      const int i = (k * GT + t) * 8;
      if (i < n) {
        load8(at + i, kept[k]);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum += kept[k][e] * kept[k][e];
      }
    }
    const int rest = (PN_KEEP * GT + t) * 8;
    for (int i = rest; i < n; i += GT * 8) {
      float f[8];
      load8(at + i, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) sum += f[e] * f[e];
    }
    sum = GT == 32 ? warp_sum(sum) : block_total(sum, red);
    const float r = 1.f / sqrtf(sum / static_cast<float>(n) + eps);
    auto finish = [&](int i, float (&f)[8]) {
      float g[8];
      load8(wp + i, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] *= r * g[e];
      store8(at + i, f);
    };
#pragma unroll
    for (int k = 0; k < PN_KEEP; ++k) {
      const int i = (k * GT + t) * 8;
      if (i < n) finish(i, kept[k]);
    }
    for (int i = rest; i < n; i += GT * 8) {
      float f[8];
      load8(at + i, f);
      finish(i, f);
    }
  }
}

// Any sizes: element i of a run is element i % vdim of a head padded to vp.  A warp takes one run.
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
part_norm_any_kernel(T* __restrict__ y, long long ld, const float* __restrict__ w, int rows, int parts, int n, int vdim, int vp, float eps) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long tasks = static_cast<long long>(rows) * parts;
  for (long long task = static_cast<long long>(blockIdx.x) * ROW_WARPS + warp; task < tasks; task += static_cast<long long>(gridDim.x) * ROW_WARPS) {
    const long long row = task / parts;
    const int part = static_cast<int>(task - row * parts);
    T* yr = y + row * ld;
    auto column = [&](int i) {
      const int c = part * n + i;
      return c / vdim * vp + c % vdim;
    };
    float sum = 0.f;
    for (int i = lane; i < n; i += 32) {
      const float v = static_cast<float>(yr[column(i)]);
      sum += v * v;
    }
    const float r = 1.f / sqrtf(warp_sum(sum) / static_cast<float>(n) + eps);
    for (int i = lane; i < n; i += 32) {
      const int c = column(i);
      yr[c] = static_cast<T>(static_cast<float>(yr[c]) * r * w[c]);
    }
  }
}

// out = a z / rms(z) + b z^2 / rms(z^2) + c z^3 / rms(z^3) + e over rows of N elements of which `count` exist (the others are
// zero).  One block per row; the first KEEP vectors of a thread stay in registers.
template <typename T, int KEEP>
__global__ void __launch_bounds__(ROW_THREADS)
poly_norm_kernel(const T* __restrict__ z, long long ldz, T* __restrict__ out, long long ldo, const float* __restrict__ coef, int rows, int N, int count,
                 float eps) {
  __shared__ float red[3][ROW_WARPS];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int row = blockIdx.x; row < rows; row += gridDim.x) {
    const T* zr = z + static_cast<long long>(row) * ldz;
    T* yr = out + static_cast<long long>(row) * ldo;
    uint4 kept[KEEP][sizeof(T) / 2];
    float s[3] = {0.f, 0.f, 0.f};
    auto add = [&](const float (&f)[8]) {
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float q = f[e] * f[e];
        s[0] += q;
        s[1] += q * q;
        s[2] += q * q * q;
      }
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = (k * ROW_THREADS + threadIdx.x) * 8;
      if (i < N) raw_load(zr + i, kept[k]);
    }
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      if ((k * ROW_THREADS + static_cast<int>(threadIdx.x)) * 8 < N) {
        float f[8];
        raw_unpack(kept[k], f);
        add(f);
      }
    }
    const int rest = (KEEP * ROW_THREADS + threadIdx.x) * 8;
    for (int i = rest; i < N; i += ROW_THREADS * 8) {
      float f[8];
      load8(zr + i, f);
      add(f);
    }
    __syncthreads();                       // the previous row's sums have been read
#pragma unroll
    for (int j = 0; j < 3; ++j) {
      s[j] = warp_sum(s[j]);
      if (lane == 0) red[j][warp] = s[j];
    }
    __syncthreads();
    float c[3];
#pragma unroll
    for (int j = 0; j < 3; ++j) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < ROW_WARPS; ++w) v += red[j][w];
      c[j] = coef[j] / sqrtf(v / static_cast<float>(count) + eps);
    }
    const float last = coef[3];
    auto finish = [&](int i, float (&f)[8]) {
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = ((c[2] * f[e] + c[1]) * f[e] + c[0]) * f[e] + last;
      store8(yr + i, f);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = (k * ROW_THREADS + threadIdx.x) * 8;
      if (i < N) {
        float f[8];
        raw_unpack(kept[k], f);
        finish(i, f);
      }
    }
    for (int i = rest; i < N; i += ROW_THREADS * 8) {
      float f[8];
      load8(zr + i, f);
      finish(i, f);
    }
  }
}

// ---------------------------------------------------------------- packed projection -> attention, per head
struct HeadFinishParams {
  void* packed;             // [rows, ld]
  long long ld;
  const int* pos;
  const int* slots;
  const int* block_table;
  void* k_cache;            // null: the layer has queries only (it reads another layer's pages)
  void* v_cache;
  const float* q_weight;    // [D]; null: no norm
  const float* k_weight;
  const float2* table;      // [positions, half]: cos, sin; null: no rotation
  int rows, q_off, Hq, k_off, v_off, Hkv, D, Dv, d_true, half, positions;
  float eps;
  int block_size, max_blocks, num_blocks;
};

// A warp owns one head of one row at a time: q heads, then k heads, then v heads.  The head goes through shared
// memory in fp32 because rotation pairs element i with i + half, in another lane.
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
qkv_head_finish_kernel(const HeadFinishParams p) {
  extern __shared__ float head_sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* s = head_sm + warp * p.D;
  const int tasks = p.Hq + (p.k_cache ? 2 * p.Hkv : 0);
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x) {
    T* y = static_cast<T*>(p.packed) + static_cast<long long>(row) * p.ld;
    const int position = p.pos[row];
    long long token = -1;
    if (p.k_cache) {
      const int blk = p.block_table[static_cast<long long>(p.slots[row]) * p.max_blocks + position / p.block_size];
      if (blk >= 0 && blk < p.num_blocks) token = static_cast<long long>(blk) * p.block_size + position % p.block_size;
    }
    const float2* cs = p.table ? p.table + static_cast<long long>(min(position, p.positions - 1)) * p.half : nullptr;
    for (int task = blockIdx.y * ROW_WARPS + warp; task < tasks; task += gridDim.y * ROW_WARPS) {
      if (task >= p.Hq + p.Hkv) {
        const int h = task - p.Hq - p.Hkv;
        if (token >= 0)
          for (int i = lane * 8; i < p.Dv; i += 256) {
            float f[8];
            load8(y + p.v_off + h * p.Dv + i, f);
            store8(static_cast<T*>(p.v_cache) + (token * p.Hkv + h) * p.Dv + i, f);
          }
        continue;
      }
      const bool is_q = task < p.Hq;
      const int h = is_q ? task : task - p.Hq;
      if (!is_q && token < 0) continue;
      T* src = y + (is_q ? p.q_off : p.k_off) + h * p.D;
      T* dst = is_q ? src : static_cast<T*>(p.k_cache) + (token * p.Hkv + h) * p.D;
      const float* w = is_q ? p.q_weight : p.k_weight;
      float sum = 0.f;
      for (int i = lane * 8; i < p.D; i += 256) {
        float f[8];
        load8(src + i, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          sum += f[e] * f[e];
          s[i + e] = f[e];
        }
      }
      float r = 1.f;
      if (w) r = 1.f / sqrtf(warp_sum(sum) / static_cast<float>(p.d_true) + p.eps);
      __syncwarp();
      for (int i = lane * 8; i < p.D; i += 256) {
        float f[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const int d = i + e;
          float v = w ? s[d] * r * w[d] : s[d];
          if (cs && d < 2 * p.half) {
            const int j = d < p.half ? d : d - p.half, o = d < p.half ? d + p.half : j;
            const float other = w ? s[o] * r * w[o] : s[o];
            const float2 t = cs[j];
            v = d < p.half ? v * t.x - other * t.y : v * t.x + other * t.y;
          }
          f[e] = v;
        }
        store8(dst + i, f);
      }
      __syncwarp();
    }
  }
}

// The same for heads of 8 * L elements, L = 4 .. 16 lanes with eight elements each, when the rotated half is a multiple of
// eight: elements stay in registers, the partner of an element lies in another lane at the same place.  A warp takes one
// item at a time: HF_BATCH times 32 / L heads of one row's queries or keys, or a run of its values.
constexpr int HF_BATCH = 2;

template <typename T, int L>
__global__ void __launch_bounds__(ROW_THREADS, 4)
qkv_head_lanes_kernel(const HeadFinishParams p) {
  constexpr int HPW = 32 / L, D = 8 * L, ITEM_HEADS = HPW * HF_BATCH, ITEM_VALUES = 256 * HF_BATCH;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, hl = lane % L, d = hl * 8;
  const bool rotated = p.table && d < 2 * p.half, first = d < p.half;
  const int j = first ? d : d - p.half;
  const int partner = (lane - hl) + (rotated ? (first ? hl + p.half / 8 : hl - p.half / 8) : hl);
  const float inv_count = 1.f / static_cast<float>(p.d_true), sign = first ? -1.f : 1.f;
  const int n_values = p.Hkv * p.Dv;
  const int q_items = (p.Hq + ITEM_HEADS - 1) / ITEM_HEADS, k_items = (p.Hkv + ITEM_HEADS - 1) / ITEM_HEADS;
  const int row_items = q_items + k_items + (n_values + ITEM_VALUES - 1) / ITEM_VALUES;
  const long long items = static_cast<long long>(p.rows) * row_items;
  for (long long item = static_cast<long long>(blockIdx.x) * ROW_WARPS + warp; item < items; item += static_cast<long long>(gridDim.x) * ROW_WARPS) {
    const int row = static_cast<int>(item / row_items), kind = static_cast<int>(item - static_cast<long long>(row) * row_items);
    T* y = static_cast<T*>(p.packed) + static_cast<long long>(row) * p.ld;
    const bool is_q = kind < q_items, is_v = kind >= q_items + k_items;
    const int h0 = (is_q ? kind : kind - q_items) * ITEM_HEADS + lane / L, heads = is_q ? p.Hq : p.Hkv;
    const int v0 = (kind - q_items - k_items) * ITEM_VALUES + lane * 8;
    const T* src = y + (is_v ? p.v_off + v0 : (is_q ? p.q_off : p.k_off) + h0 * D + d);
    const int step = is_v ? 256 : HPW * D;
    float v[HF_BATCH][8];
    bool ok[HF_BATCH];
#pragma unroll
    for (int i = 0; i < HF_BATCH; ++i) {           // what does not depend on the position is asked for first
      ok[i] = is_v ? v0 + i * 256 < n_values : h0 + i * HPW < heads;
      if (ok[i]) load8(src + i * step, v[i]);
      else
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] = 0.f;
    }
    const int position = p.pos[row];
    long long token = 0;
    if (!is_q) {
      const int blk = p.block_table[static_cast<long long>(p.slots[row]) * p.max_blocks + position / p.block_size];
      if (blk < 0 || blk >= p.num_blocks) continue;
      token = static_cast<long long>(blk) * p.block_size + position % p.block_size;
    }
    if (is_v) {
#pragma unroll
      for (int i = 0; i < HF_BATCH; ++i)
        if (ok[i]) store8(static_cast<T*>(p.v_cache) + token * n_values + v0 + i * 256, v[i]);
      continue;
    }
    float cs[8], sn[8], w[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) { cs[e] = w[e] = 1.f; sn[e] = 0.f; }
    if (rotated) {
      const float4* t = reinterpret_cast<const float4*>(p.table + static_cast<long long>(min(position, p.positions - 1)) * p.half + j);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float4 a = __ldg(t + e);
        cs[2 * e] = a.x; cs[2 * e + 1] = a.z;
        sn[2 * e] = sign * a.y; sn[2 * e + 1] = sign * a.w;
      }
    }
    const float* weight = is_q ? p.q_weight : p.k_weight;
    if (weight) load8(weight + d, w);
    T* dst = is_q ? y + p.q_off + h0 * D + d : static_cast<T*>(p.k_cache) + (token * p.Hkv + h0) * D + d;
#pragma unroll
    for (int i = 0; i < HF_BATCH; ++i) {
      float r = 1.f;
      if (weight) {                                 // the same in every lane of the warp
        float sum = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) sum += v[i][e] * v[i][e];
#pragma unroll
        for (int o = L / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        r = rsqrtf(sum * inv_count + p.eps);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) v[i][e] *= r * w[e];
      if (p.table) {
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const float other = __shfl_sync(0xffffffffu, v[i][e], partner);
          v[i][e] = v[i][e] * cs[e] + other * sn[e];
        }
      }
      if (ok[i]) store8(dst + i * step, v[i]);
    }
  }
}

}  // namespace ft

using namespace ft;

static bool row_aligned(std::initializer_list<const void*> ps) {
  uintptr_t v = 0;
  for (const void* p : ps) v |= reinterpret_cast<uintptr_t>(p);
  return (v & 15) == 0;
}

// y[rows, H] (bf16, or fp32 with out_f32) = RMS norm of x rows times (offset + w).  x: fp32, or bf16 with in_bf16,
// [n_src, ldx]; ids (int64 [rows] or null): the rows to take.  terms ([term_rows, ldt], type of y) and where (int32
// [n_src, n_terms]; entries outside 0 .. term_rows - 1 add nothing): added to the row first.  x_out: fp32 [rows,
// ldo] receives the row with its terms, and may be x when ids is null.  count: true width (padding is zero).
FT_API int ft_rms_rows(const void* x, const long long* ids, int n_src, int in_bf16, float* x_out, const void* terms,
                       const int* where, int n_terms, int term_rows, const float* w, void* y, int out_f32, int rows, int H,
                       int count, long long ldx, long long ldo, long long ldt, long long ldy, float eps, float offset,
                       int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(x && w && y, "ft_rms_rows: null pointer");
  FT_REQUIRE(H > 0 && H % 8 == 0 && count > 0 && count <= H && ((ldx | ldo | ldt | ldy) & 7) == 0 && ldx >= H && ldy >= H,
             "ft_rms_rows: H=%d and strides must be multiples of 8", H);
  FT_REQUIRE(n_terms == 0 || (terms && where && n_terms > 0 && ldt >= H && term_rows > 0), "ft_rms_rows: terms without their rows");
  FT_REQUIRE(!x_out || ldo >= H, "ft_rms_rows: row stride of the residual");
  FT_REQUIRE(row_aligned({x, x_out, terms, w, y}), "ft_rms_rows: pointers must be 16-byte aligned");
  FT_REQUIRE(n_src > 0 && (ids || rows <= n_src), "ft_rms_rows: %d source rows", n_src);
  if (rows <= 0) return FT_E_OK;
  RmsRowsParams p;
  p.x = x; p.ids = ids; p.x_out = x_out; p.terms = terms; p.where = where; p.w = w; p.y = y;
  p.ldx = ldx; p.ldo = ldo; p.ldt = ldt; p.ldy = ldy;
  p.rows = rows; p.n_src = n_src; p.H = H; p.count = count; p.n_terms = n_terms; p.term_rows = term_rows;
  p.eps = eps; p.offset = offset;
  const int cap = sm_count(device) * 32;
  const int grid = rows < cap ? rows : cap;
  if (in_bf16) {
    if (out_f32) rms_rows_kernel<__nv_bfloat16, float><<<grid, ROW_THREADS, 0, stream>>>(p);
    else rms_rows_kernel<__nv_bfloat16, __nv_bfloat16><<<grid, ROW_THREADS, 0, stream>>>(p);
  } else {
    if (out_f32) rms_rows_kernel<float, float><<<grid, ROW_THREADS, 0, stream>>>(p);
    else rms_rows_kernel<float, __nv_bfloat16><<<grid, ROW_THREADS, 0, stream>>>(p);
  }
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// x' = norm(alpha x + sigmoid(gate) (dense_weight dense + sum_j weight_j terms[where_j])) * w for `n_rows` rows (see SumNormParams), RMS
// over `count` elements, into x_out and, as bf16 or with out_f32 as fp32, into h; with w2 h goes through a second norm.  x: fp32, or
// bf16 with in_bf16 (fp32 embeddings: in_bf16 0).  dense, terms and gate have the type of h.  H and strides multiples of 8.
FT_API int ft_sum_norm_rows(const void* x, long long ldx, const long long* ids, int n_src, int in_bf16, const long long* rows, const void* dense,
                            long long ldd, const float* dense_weight, const void* terms, long long ldt, int term_rows, const int* where,
                            const float* weight, int n_terms, const void* gate, long long ldg, float alpha, const float* w, const float* w2,
                            float* x_out, long long ldo, void* h, long long ldh, int out_f32, int n_rows, int tokens, int H, int count,
                            float eps, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(x && w && (x_out || h) && (dense || n_terms > 0), "ft_sum_norm_rows: null pointer");
  FT_REQUIRE(H > 0 && H % 8 == 0 && count > 0 && count <= H && ((ldx | ldd | ldt | ldg | ldo | ldh) & 7) == 0 && ldx >= H,
             "ft_sum_norm_rows: H=%d and strides must be multiples of 8", H);
  FT_REQUIRE(n_terms == 0 || (terms && where && n_terms > 0 && ldt >= H && term_rows > 0), "ft_sum_norm_rows: terms without their rows");
  FT_REQUIRE((!dense || ldd >= H) && (!gate || ldg >= H) && (!x_out || ldo >= H) && (!h || ldh >= H), "ft_sum_norm_rows: row strides");
  FT_REQUIRE(row_aligned({x, dense, terms, gate, w, w2, x_out, h}), "ft_sum_norm_rows: pointers must be 16-byte aligned");
  FT_REQUIRE(n_src > 0 && (ids || tokens <= n_src) && (rows || n_rows <= tokens), "ft_sum_norm_rows: %d source rows", n_src);
  FT_REQUIRE(x_out != x || (!ids && !rows && !in_bf16), "ft_sum_norm_rows: gathered rows cannot be updated in place");
  if (n_rows <= 0) return FT_E_OK;
  SumNormParams p;
  p.x = x; p.ids = ids; p.rows = rows; p.dense = dense; p.dense_weight = dense_weight; p.terms = terms; p.where = where; p.weight = weight;
  p.gate = gate; p.w = w; p.w2 = w2; p.x_out = x_out; p.h = h;
  p.ldx = ldx; p.ldd = ldd; p.ldt = ldt; p.ldg = ldg; p.ldo = ldo; p.ldh = ldh;
  p.n_rows = n_rows; p.tokens = tokens; p.n_src = n_src; p.H = H; p.count = count; p.n_terms = n_terms; p.term_rows = term_rows;
  p.alpha = alpha; p.eps = eps;
  const int cap = sm_count(device) * 32;
  const int grid = n_rows < cap ? n_rows : cap;
  if (in_bf16) {
    if (out_f32) sum_norm_rows_kernel<__nv_bfloat16, float><<<grid, ROW_THREADS, 0, stream>>>(p);
    else sum_norm_rows_kernel<__nv_bfloat16, __nv_bfloat16><<<grid, ROW_THREADS, 0, stream>>>(p);
  } else {
    if (out_f32) sum_norm_rows_kernel<float, float><<<grid, ROW_THREADS, 0, stream>>>(p);
    else sum_norm_rows_kernel<float, __nv_bfloat16><<<grid, ROW_THREADS, 0, stream>>>(p);
  }
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// RMS norm, in place, of `parts` equal runs of rows y [rows, ld] on their own, times w [heads * vp].  A row is heads of vdim
// elements padded to vp; runs count the elements that exist.  bf16, or fp32 with f32.
FT_API int ft_part_norm(void* y, long long ld, const float* w, int rows, int heads, int vdim, int vp, int parts, float eps, int f32, int device,
                        cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(y && w, "ft_part_norm: null pointer");
  const long long inner = static_cast<long long>(heads) * vdim;
  FT_REQUIRE(heads > 0 && vdim > 0 && vp >= vdim && parts > 0 && inner % parts == 0 && static_cast<long long>(heads) * vp < (1ll << 31) &&
                 ld >= static_cast<long long>(heads) * vp, "ft_part_norm: %d heads of %d in %d parts", heads, vdim, parts);
  if (rows <= 0) return FT_E_OK;
  const int n = static_cast<int>(inner / parts), cap = sm_count(device) * 16;
  const bool vectors = vp == vdim && n % 8 == 0 && ld % 8 == 0 && row_aligned({y, w});
  const bool wide = vectors && n > PN_KEEP * 256;
  const long long tasks = static_cast<long long>(rows) * parts, need = wide ? tasks : (tasks + ROW_WARPS - 1) / ROW_WARPS;
  const int grid = need < cap ? static_cast<int>(need) : cap;
#define FT_PN(T)                                                                                                        \
  if (wide) part_norm_kernel<T, 256><<<grid, ROW_THREADS, 0, stream>>>(static_cast<T*>(y), ld, w, rows, parts, n, eps);  \
  else if (vectors) part_norm_kernel<T, 32><<<grid, ROW_THREADS, 0, stream>>>(static_cast<T*>(y), ld, w, rows, parts, n, eps); \
  else part_norm_any_kernel<T><<<grid, ROW_THREADS, 0, stream>>>(static_cast<T*>(y), ld, w, rows, parts, n, vdim, vp, eps);
  if (f32) { FT_PN(float) } else { FT_PN(__nv_bfloat16) }
#undef FT_PN
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// out [rows, N] = a N(z) + b N(z^2) + c N(z^3) + e with coef = (a, b, c, e) fp32, N dividing a row by its root mean square over `count`
// elements (those behind them are zero; they become e).  bf16, or fp32 with f32; N and strides multiples of 8.
FT_API int ft_poly_norm(const void* z, long long ldz, void* out, long long ldo, const float* coef, int rows, int N, int count, float eps, int f32,
                        int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(z && out && coef, "ft_poly_norm: null pointer");
  FT_REQUIRE(N > 0 && N % 8 == 0 && count > 0 && count <= N && ldz >= N && ldo >= N && ((ldz | ldo) & 7) == 0 && row_aligned({z, out}),
             "ft_poly_norm: N=%d and strides must be multiples of 8", N);
  if (rows <= 0) return FT_E_OK;
  const int cap = sm_count(device) * 16, grid = rows < cap ? rows : cap;
#define FT_PO(T, K) \
  poly_norm_kernel<T, K><<<grid, ROW_THREADS, 0, stream>>>(static_cast<const T*>(z), ldz, static_cast<T*>(out), ldo, coef, rows, N, count, eps)
  if (f32) FT_PO(float, 4);
  else if (N <= 2 * ROW_THREADS * 8) FT_PO(__nv_bfloat16, 2);
  else if (N <= 6 * ROW_THREADS * 8) FT_PO(__nv_bfloat16, 6);
  else FT_PO(__nv_bfloat16, 12);
#undef FT_PO
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// The pass between a packed projection and its attention (see qkv_head_finish_kernel).  packed and caches are bf16, or
// fp32 with f32; offsets in elements, multiples of 8; head sizes D / Dv multiples of 8 of which d_true elements of a q
// or k head exist (padding is zero).  k_cache null: no keys and values in the row.  table: fp32 pairs (cos, sin)
// [positions, half] or null.
FT_API int ft_qkv_head_finish(void* packed, long long ld, const int* pos, const int* slots, const int* block_table,
                              void* k_cache, void* v_cache, const float* q_weight, const float* k_weight, const void* table,
                              int rows, int q_off, int Hq, int k_off, int v_off, int Hkv, int D, int Dv, int d_true, int half,
                              int positions, float eps, int f32, int block_size, int max_blocks, int num_blocks, int device,
                              cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(packed && pos && (!k_cache || (v_cache && slots && block_table)), "ft_qkv_head_finish: null pointer");
  FT_REQUIRE(((q_off | k_off | v_off | D | Dv) & 7) == 0 && ld % 8 == 0, "ft_qkv_head_finish: offsets, sizes and strides must be multiples of 8");
  FT_REQUIRE(Hq > 0 && D > 0 && D <= 1024 && d_true > 0 && d_true <= D && q_off >= 0 && q_off + static_cast<long long>(Hq) * D <= ld,
             "ft_qkv_head_finish: the queries lie outside the row");
  FT_REQUIRE(!k_cache || (Hkv > 0 && Dv > 0 && k_off >= 0 && v_off >= 0 && k_off + static_cast<long long>(Hkv) * D <= ld &&
                          v_off + static_cast<long long>(Hkv) * Dv <= ld && block_size > 0 && max_blocks > 0 && num_blocks > 0),
             "ft_qkv_head_finish: the keys or values lie outside the row");
  FT_REQUIRE(!table || (half > 0 && 2 * half <= d_true && positions > 0), "ft_qkv_head_finish: rotation of %d elements of %d", 2 * half, d_true);
  FT_REQUIRE(row_aligned({packed, k_cache, v_cache}) && (reinterpret_cast<uintptr_t>(table) & 7) == 0,
             "ft_qkv_head_finish: pointers must be 16-byte aligned");
  if (rows <= 0) return FT_E_OK;
  HeadFinishParams p;
  p.packed = packed; p.ld = ld; p.pos = pos; p.slots = slots; p.block_table = block_table;
  p.k_cache = k_cache; p.v_cache = v_cache; p.q_weight = q_weight; p.k_weight = k_weight;
  p.table = static_cast<const float2*>(table);
  p.rows = rows; p.q_off = q_off; p.Hq = Hq; p.k_off = k_off; p.v_off = v_off; p.Hkv = k_cache ? Hkv : 0;
  p.D = D; p.Dv = Dv; p.d_true = d_true; p.half = half; p.positions = positions; p.eps = eps;
  p.block_size = block_size; p.max_blocks = max_blocks; p.num_blocks = num_blocks;
  const int wave = sm_count(device) * 8;
  if ((D == 32 || D == 64 || D == 128) && (!table || (half % 8 == 0 && (reinterpret_cast<uintptr_t>(table) & 15) == 0)) &&
      row_aligned({q_weight, k_weight})) {
    const int per_pass = 32 / (D / 8) * HF_BATCH;
    const long long items = static_cast<long long>(rows) * ((Hq + per_pass - 1) / per_pass + (p.Hkv + per_pass - 1) / per_pass +
                                                            (p.Hkv * Dv + 256 * HF_BATCH - 1) / (256 * HF_BATCH));
    const long long need = (items + ROW_WARPS - 1) / ROW_WARPS;
    const int grid = need < 4 * wave ? static_cast<int>(need) : 4 * wave;
#define FT_HL(T, LL) qkv_head_lanes_kernel<T, LL><<<grid, ROW_THREADS, 0, stream>>>(p)
    if (f32) {
      if (D == 32) FT_HL(float, 4); else if (D == 64) FT_HL(float, 8); else FT_HL(float, 16);
    } else {
      if (D == 32) FT_HL(__nv_bfloat16, 4); else if (D == 64) FT_HL(__nv_bfloat16, 8); else FT_HL(__nv_bfloat16, 16);
    }
#undef FT_HL
    FT_CUDA_CHECK(cudaGetLastError());
    count_launch();
    return FT_E_OK;
  }
  // heads of a row are spread over blocks when the rows alone do not fill the GPU
  const int tasks = Hq + 2 * p.Hkv;
  int parts = (tasks + ROW_WARPS - 1) / ROW_WARPS;
  if (parts > wave / rows) parts = wave / rows > 1 ? wave / rows : 1;
  const dim3 grid(rows < wave ? rows : wave, parts);
  const size_t smem = static_cast<size_t>(ROW_WARPS) * D * sizeof(float);
  if (f32) qkv_head_finish_kernel<float><<<grid, ROW_THREADS, smem, stream>>>(p);
  else qkv_head_finish_kernel<__nv_bfloat16><<<grid, ROW_THREADS, smem, stream>>>(p);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}
