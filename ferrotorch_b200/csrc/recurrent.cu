// Recurrent decoder blocks: short causal convolutions with carried inputs, and linear recurrences over prompt portions.
//
//   ft_causal_conv   per channel, over the rows of a ragged batch, with or without a silu of the result; the inputs ahead of
//                    a portion come from the sequence's slot, the rows that are a sequence's only token store their own
//                    inputs there
//   ft_conv_tail     the last inputs of portions into the slots, where no scan follows that does it
//   ft_rglru_scan    S_t = a_t S_(t-1) + x_t over the rows of every portion, out = S * gelu(y); the final state and
//                    the convolution's last inputs go to the slot
//
// A slot needs no clearing: what a sequence has seen follows from its positions, and position 0 starts from zero.
#include <initializer_list>

#include "recurrent.cuh"

namespace ft {

constexpr int CV_THREADS = 128;
constexpr int CV_BATCH = 4;      // rows loaded together
constexpr int CV_ROWS = 16;      // most consecutive rows a thread walks (their inputs overlap)

struct ConvParams {
  const void* x;            // [rows, ldx]
  const float* w;           // [taps, C]: w[taps - 1] weighs the row itself
  const float* bias;        // [C]
  void* state;              // [slots, taps - 1, C]: the last inputs of a sequence, the most recent one last
  void* u;                  // [rows, ldu]
  const int* pos;
  const int* slots;
  const int* starts;        // position of the first row of the row's portion
  long long ldx, ldu;
  int rows, n_single, C, taps, walk, silu;
};

// The result of a channel: the sum itself or its silu (in the form of the type, see recurrent.cuh).
template <typename T>
__device__ __forceinline__ void conv_finish(const ConvParams& p, float (&v)[8]) {
  if (!p.silu) return;
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] *= sigmoid_row(v[e], static_cast<const T*>(nullptr));
}

// The input d rows ahead of a row (d <= taps - 1): of the same portion, of the slot, or zero ahead of the sequence.
template <typename T>
__device__ __forceinline__ void conv_input(const ConvParams& p, const T* x, const T* st, int row, int pos, int back, int d, float (&v)[8]) {
  if (pos - d < 0) {
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = 0.f;
  } else if (d <= back) {
    load8(x + static_cast<long long>(row - d) * p.ldx, v);
  } else {
    load8(st + static_cast<long long>(p.taps - 1 - (d - back)) * p.C, v);
  }
}

// Up to four taps: weights and the sliding inputs stay in registers while the thread walks down its rows.
template <typename T, int TAPS>
__global__ void __launch_bounds__(CV_THREADS, 5)
short_conv_kernel(const ConvParams p) {
  const int c = (blockIdx.x * CV_THREADS + threadIdx.x) * 8;
  if (c >= p.C) return;
  float w[TAPS][8], bias[8], in[TAPS][8];      // in[d]: the input d rows ahead
  load8(p.bias + c, bias);
#pragma unroll
  for (int d = 0; d < TAPS; ++d) load8(p.w + static_cast<long long>(TAPS - 1 - d) * p.C + c, w[d]);
  const T* x = static_cast<const T*>(p.x) + c;
  for (int r0 = blockIdx.y * p.walk; r0 < p.rows; r0 += gridDim.y * p.walk) {
    const int r1 = min(r0 + p.walk, p.rows);
    for (int rb = r0; rb < r1; rb += CV_BATCH) {
      float now[CV_BATCH][8];
      int pos[CV_BATCH], back[CV_BATCH];
#pragma unroll
      for (int i = 0; i < CV_BATCH; ++i) {     // past the end: the last row again
        const int row = min(rb + i, r1 - 1);
        load8(x + static_cast<long long>(row) * p.ldx, now[i]);
        pos[i] = __ldg(p.pos + row);
        back[i] = pos[i] - __ldg(p.starts + row);
      }
#pragma unroll
      for (int i = 0; i < CV_BATCH; ++i) {
        const int row = rb + i;
        if (row >= r1) break;
        const bool single = row < p.n_single;
        T* st = static_cast<T*>(p.state);
        if (single || back[i] < TAPS - 1) st += static_cast<long long>(p.slots[row]) * (TAPS - 1) * p.C + c;
        if (row == r0 || back[i] == 0) {       // a walk or a portion begins: fetch what lies ahead of this row
#pragma unroll
          for (int d = 1; d < TAPS; ++d) conv_input(p, x, static_cast<const T*>(st), row, pos[i], back[i], d, in[d]);
        }
        float acc[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) { in[0][e] = now[i][e]; acc[e] = bias[e]; }
#pragma unroll
        for (int d = TAPS - 1; d >= 0; --d)
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[e] += w[d][e] * in[d][e];
        conv_finish<T>(p, acc);
        store8(static_cast<T*>(p.u) + static_cast<long long>(row) * p.ldu + c, acc);
        if (TAPS > 1 && single) {              // this thread is the only one at these inputs
#pragma unroll
          for (int d = 0; d < TAPS - 1; ++d) store8(st + static_cast<long long>(TAPS - 2 - d) * p.C, in[d]);
        }
#pragma unroll
        for (int d = TAPS - 1; d > 0; --d)
#pragma unroll
          for (int e = 0; e < 8; ++e) in[d][e] = in[d - 1][e];
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(CV_THREADS)
causal_conv_kernel(const ConvParams p) {
  const int c = (blockIdx.x * CV_THREADS + threadIdx.x) * 8;
  if (c >= p.C) return;
  const int keep = p.taps - 1;
  float bias[8];
  load8(p.bias + c, bias);
  const T* x = static_cast<const T*>(p.x) + c;
  for (int r0 = blockIdx.y * p.walk; r0 < p.rows; r0 += gridDim.y * p.walk)
    for (int row = r0; row < min(r0 + p.walk, p.rows); ++row) {
      const int pos = p.pos[row], back = pos - p.starts[row];       // rows of this portion ahead of this one
      T* st = static_cast<T*>(p.state) + static_cast<long long>(p.slots[row]) * keep * p.C + c;
      float acc[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] = bias[e];
      for (int d = keep; d >= 0; --d) {
        float v[8], w[8];
        conv_input(p, x, static_cast<const T*>(st), row, pos, back, d, v);
        load8(p.w + static_cast<long long>(keep - d) * p.C + c, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] += w[e] * v[e];
      }
      conv_finish<T>(p, acc);
      store8(static_cast<T*>(p.u) + static_cast<long long>(row) * p.ldu + c, acc);
      if (row < p.n_single) {                                       // this thread is the only one at these inputs
        float v[8];
        for (int m = 0; m + 1 < keep; ++m) {
          load8(static_cast<const T*>(st) + static_cast<long long>(m + 1) * p.C, v);
          store8(st + static_cast<long long>(m) * p.C, v);
        }
        if (keep > 0) {
          load8(x + static_cast<long long>(row) * p.ldx, v);
          store8(st + static_cast<long long>(keep - 1) * p.C, v);
        }
      }
    }
}

// The last `keep` inputs of every portion into its slot: from the portion, or what the slot held (moved down; m + n > m is still
// old).  A thread owns eight channels.
template <typename T>
__global__ void __launch_bounds__(CV_THREADS)
conv_tail_kernel(const T* __restrict__ x, long long ldx, T* state, const int* __restrict__ spans, int C, int keep) {
  const int c = (blockIdx.x * CV_THREADS + threadIdx.x) * 8;
  if (c >= C) return;
  const int* span = spans + 4 * blockIdx.y;
  const int slot = span[0], row0 = span[1], n = span[3];
  T* st = state + static_cast<long long>(slot) * keep * C + c;
  for (int m = 0; m < keep; ++m) {
    const int o = n - keep + m;
    float v[8];
    if (o >= 0) load8(x + static_cast<long long>(row0 + o) * ldx + c, v);
    else load8(static_cast<const T*>(st) + static_cast<long long>(m + n) * C, v);
    store8(st + static_cast<long long>(m) * C, v);
  }
}

// ---------------------------------------------------------------- scan
// One block per (32 channels, portion): lane = channel, a warp takes SC_STEP consecutive rows of a tile of
// SC_WARPS * SC_STEP.  Every warp folds its rows into (product of decays, state from zero), the folds of a tile are
// combined through shared memory, then every warp walks its rows again from its true state.  Each input is read once;
// the next tile is loaded while one is computed.
constexpr int SC_WARPS = 8;
constexpr int SC_STEP = 8;

struct ScanParams {
  const float* a;           // [rows, C]
  const float* x;
  const void* y;            // [rows, ldy]: the other branch
  void* out;                // [rows, ldo]
  float* state;             // [slots, C]
  const int* spans;         // [n, 4]: slot, first row, first position, rows
  const void* conv_x;       // [rows, ldc] inputs of the convolution, and its state (null: no convolution)
  void* conv_state;
  long long ldy, ldo, ldc;
  int C, keep;
};

template <typename T>
__global__ void __launch_bounds__(SC_WARPS * 32, 3)
rglru_scan_kernel(const ScanParams p) {
  __shared__ float fold_a[2][SC_WARPS][32], fold_s[2][SC_WARPS][32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x * 32 + lane;
  const bool c_ok = c < p.C;
  const int cc = c_ok ? c : p.C - 1;
  const int* span = p.spans + 4 * blockIdx.y;
  const int slot = span[0], row0 = span[1], pos0 = span[2], n = span[3];
  float* st = p.state + static_cast<long long>(slot) * p.C + cc;
  float a[SC_STEP], x[SC_STEP];
  T y[SC_STEP];
  // every load is issued (past the end: of the last row), so that all of a tile are in flight together
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < SC_STEP; ++i) {
      const long long row = row0 + min(t0 + i, n - 1);
      a[i] = __ldg(p.a + row * p.C + cc);
      x[i] = __ldg(p.x + row * p.C + cc);
      y[i] = static_cast<const T*>(p.y)[row * p.ldy + cc];
    }
  };
  fetch(warp * SC_STEP);
  float carry = pos0 == 0 ? 0.f : *st;
  int buf = 0;
  for (int base = 0; base < n; base += SC_WARPS * SC_STEP, buf ^= 1) {
    const int t0 = base + warp * SC_STEP;
    float ca[SC_STEP], cx[SC_STEP];
    T cy[SC_STEP];
    float fa = 1.f, fs = 0.f;
#pragma unroll
    for (int i = 0; i < SC_STEP; ++i) {
      const bool ok = t0 + i < n;
      ca[i] = ok ? a[i] : 1.f;
      cx[i] = ok ? x[i] : 0.f;
      cy[i] = y[i];
      fs = ca[i] * fs + cx[i];
      fa *= ca[i];
    }
    if (base + SC_WARPS * SC_STEP < n) fetch(t0 + SC_WARPS * SC_STEP);
    fold_a[buf][warp][lane] = fa;
    fold_s[buf][warp][lane] = fs;
    __syncthreads();          // one barrier per tile: the next tile folds into the other buffer
    float s = carry;
#pragma unroll
    for (int w = 0; w < SC_WARPS; ++w) {
      const float next = fold_a[buf][w][lane] * carry + fold_s[buf][w][lane];
      if (w < warp) s = next;
      carry = next;
    }
#pragma unroll
    for (int i = 0; i < SC_STEP; ++i) {
      s = ca[i] * s + cx[i];
      if (t0 + i < n && c_ok)
        static_cast<T*>(p.out)[(row0 + t0 + i) * p.ldo + c] = static_cast<T>(s * gelu_row(static_cast<float>(cy[i]), static_cast<const T*>(nullptr)));
    }
  }
  if (warp == 0 && c_ok) *st = carry;
  if (warp == SC_WARPS - 1 && c_ok && p.conv_state) {
    // the last inputs of the sequence: from this portion, or what the slot held (moved down; m + n > m is still old)
    T* cs = static_cast<T*>(p.conv_state) + static_cast<long long>(slot) * p.keep * p.C + c;
    for (int m = 0; m < p.keep; ++m) {
      const int o = n - p.keep + m;
      cs[static_cast<long long>(m) * p.C] = o >= 0 ? static_cast<const T*>(p.conv_x)[(row0 + o) * p.ldc + c]
                                                   : cs[static_cast<long long>(m + n) * p.C];
    }
  }
}

static bool rc_aligned(std::initializer_list<const void*> ps) {
  uintptr_t v = 0;
  for (const void* p : ps) v |= reinterpret_cast<uintptr_t>(p);
  return (v & 15) == 0;
}

}  // namespace ft

using namespace ft;

// u = causal convolution of x over the rows of a ragged batch (see ConvParams).  x, state and u are bf16, or fp32
// with f32; w [taps, C] and bias [C] fp32; C a multiple of 8.  silu: of the result.
FT_API int ft_causal_conv(const void* x, long long ldx, const float* w, const float* bias, void* state, void* u, long long ldu,
                          const int* pos, const int* slots, const int* starts, int rows, int n_single, int C, int taps, int silu, int f32,
                          int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(x && w && bias && u && pos && slots && starts && (state || taps == 1), "ft_causal_conv: null pointer");
  FT_REQUIRE(C > 0 && C % 8 == 0 && taps >= 1 && ((ldx | ldu) & 7) == 0 && ldx >= C && ldu >= C, "ft_causal_conv: %d channels, %d taps", C, taps);
  FT_REQUIRE(rc_aligned({x, w, bias, state, u}) && n_single >= 0 && n_single <= rows, "ft_causal_conv: pointers must be 16-byte aligned");
  if (rows <= 0) return FT_E_OK;
  ConvParams p;
  p.x = x; p.w = w; p.bias = bias; p.state = state; p.u = u; p.pos = pos; p.slots = slots; p.starts = starts;
  p.ldx = ldx; p.ldu = ldu; p.rows = rows; p.n_single = n_single; p.C = C; p.taps = taps; p.silu = silu;
  const int gx = (C / 8 + CV_THREADS - 1) / CV_THREADS;
  p.walk = rows / (sm_count(device) * 8 / gx + 1);         // enough blocks for the GPU, then longer walks
  p.walk = p.walk < 1 ? 1 : (p.walk > CV_ROWS ? CV_ROWS : p.walk);
  const int need = (rows + p.walk - 1) / p.walk;
  const dim3 grid(gx, need < 65535 ? need : 65535);
#define FT_CONV(T)                                                                    \
  switch (taps) {                                                                     \
    case 1: short_conv_kernel<T, 1><<<grid, CV_THREADS, 0, stream>>>(p); break;       \
    case 2: short_conv_kernel<T, 2><<<grid, CV_THREADS, 0, stream>>>(p); break;       \
    case 3: short_conv_kernel<T, 3><<<grid, CV_THREADS, 0, stream>>>(p); break;       \
    case 4: short_conv_kernel<T, 4><<<grid, CV_THREADS, 0, stream>>>(p); break;       \
    default: causal_conv_kernel<T><<<grid, CV_THREADS, 0, stream>>>(p);               \
  }
  if (f32) { FT_CONV(float) } else { FT_CONV(__nv_bfloat16) }
#undef FT_CONV
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// The last `keep` rows of x [rows, ldx] of every portion (spans int32 [n_spans, 4]: slot, first row, first position, rows) into state
// [slots, keep, C].  bf16, or fp32 with f32; C a multiple of 8.
FT_API int ft_conv_tail(const void* x, long long ldx, void* state, const int* spans, int n_spans, int C, int keep, int f32, int device,
                        cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(x && state && spans, "ft_conv_tail: null pointer");
  FT_REQUIRE(C > 0 && C % 8 == 0 && keep > 0 && ldx >= C && ldx % 8 == 0 && n_spans < 65536 && rc_aligned({x, state}), "ft_conv_tail: %d channels", C);
  if (n_spans <= 0) return FT_E_OK;
  const dim3 grid((C / 8 + CV_THREADS - 1) / CV_THREADS, n_spans);
  if (f32) conv_tail_kernel<float><<<grid, CV_THREADS, 0, stream>>>(static_cast<const float*>(x), ldx, static_cast<float*>(state), spans, C, keep);
  else conv_tail_kernel<__nv_bfloat16><<<grid, CV_THREADS, 0, stream>>>(static_cast<const __nv_bfloat16*>(x), ldx, static_cast<__nv_bfloat16*>(state), spans, C, keep);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// The recurrence over n_spans portions (spans int32 [n_spans, 4]: slot, first row, first position, rows): a, x fp32
// [rows, C], y / out [rows, ldy / ldo], state fp32 [slots, C].  conv_x [rows, ldc] and conv_state [slots, keep, C]: the
// inputs of the block's convolution, whose last `keep` are stored (null: none).  bf16, or fp32 with f32.
FT_API int ft_rglru_scan(const float* a, const float* x, const void* y, long long ldy, void* out, long long ldo, float* state,
                         const int* spans, int n_spans, const void* conv_x, long long ldc, void* conv_state, int keep, int C,
                         int f32, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(a && x && y && out && state && spans, "ft_rglru_scan: null pointer");
  FT_REQUIRE(C > 0 && ldy >= C && ldo >= C && (!conv_state || (conv_x && keep >= 0 && ldc >= C)), "ft_rglru_scan: bad shape");
  if (n_spans <= 0) return FT_E_OK;
  FT_REQUIRE(n_spans < 65536, "ft_rglru_scan: %d portions", n_spans);
  ScanParams p;
  p.a = a; p.x = x; p.y = y; p.out = out; p.state = state; p.spans = spans;
  p.conv_x = conv_x; p.conv_state = keep > 0 ? conv_state : nullptr; p.ldy = ldy; p.ldo = ldo; p.ldc = ldc; p.C = C; p.keep = keep;
  const dim3 grid((C + 31) / 32, n_spans);
  if (f32) rglru_scan_kernel<float><<<grid, SC_WARPS * 32, 0, stream>>>(p);
  else rglru_scan_kernel<__nv_bfloat16><<<grid, SC_WARPS * 32, 0, stream>>>(p);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}
