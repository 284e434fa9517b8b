// Recurrences whose state is a matrix per head, S [dim, vdim], and changes by outer products k v^T.  Two rules:
//
// MEMORY, the recurrence of xLSTM's mLSTM: S and a normaliser n [dim], both relative to a running maximum m of the logarithmic gates,
//
//   i = cap tanh((zi + bi) / cap),  f = logsigmoid(cap tanh((zf + bf) / cap))
//   m' = max(f + m, i),  S' = e^(f + m - m') S + e^(i - m') k v^T,  n' likewise with k alone
//   o = S'^T q / (max(|n'.q|, e^-m') + 1e-6)
//
// followed by an RMS norm of every head's o, a weight, the sigmoid of an output gate and a constant factor.
//
// STATE_SPACE, state-space duality (Mamba-2): with step sizes dt = softplus(z + b) and a rate per head,
//
//   S' = e^(-rate dt) S + dt k v^T,  o = (S'^T q + skip v) silu(gate)
//
// where k, q (B and C there) are shared by the heads of a group.
//
// Gates, step sizes, states and all arithmetic of the recurrence are fp32; q, k, v and the output gate come from packed rows.
//
//   ft_memory_steps, ft_state_steps    token by token: rows that are their sequence's only token, short portions, any sizes,
//                                      bf16 or fp32
//   ft_memory_chunks, ft_state_chunks  whole portions in chunks of 128 tokens on tcgen05 / TMEM (bf16, dim up to 128, vdim up
//                                      to 256)
//
// Chunks.  Let b_t be the sum of f over a chunk's tokens up to t, a_t = i_t - b_t, M the maximum before the chunk and x_t =
// max(M, a_1 .. a_t).  Then m_t = b_t + x_t and
//   S_t = e^(M - x_t) S + sum_(s <= t) e^(a_s - x_t) k_s v_s^T,
// so a chunk's outputs are a causal product of scores like attention's plus q times the state at its start, and its
// contribution to the next state is one product over its tokens, independent of all other chunks.  With b the sum of -rate dt, a =
// log dt - b, x = -b and M = 0 this is the state-space rule, whose exponents never are positive where they count.  Four passes:
//   memory_gates_kernel   a, x, e^-m of every token and M of every chunk (fp32; a warp scans a chunk)
//   memory_update_kernel  U = sum_s e^(a_s - x_end) k_s v_s^T of every (chunk, head): tcgen05 product with the weighted keys
//                         as high and low bf16 halves, so that the state keeps about 16 bits more than its operands
//   memory_carry_kernel   S' = e^(M - x_end) S + U over the chunks of a portion, element by element in fp32; leaves every
//                         chunk's starting state as high and low bf16 halves and the final one in the slot
//   memory_output_kernel  O = q S, scaled row by row with e^(M - x_t) in TMEM, then + P V with the weights P = causal
//                         e^(a_s - x_t) q.k written over the scores; denominator, norm, gate and store.  S and P are operands in
//                         high and low halves: o is normed, so where keys nearly cancel, the error of a plain bf16 weight would grow.
//                         STATE_SPACE adds skip times the token's own v, which is still in shared memory
//
// A slot needs no clearing: what a sequence has seen follows from its positions, and position 0 starts from zero.
#include <initializer_list>

#include "row_vec.cuh"

namespace ft {

enum : int { MEMORY = 0, STATE_SPACE = 1 };

struct MemoryParams {
  const void* q;            // packed rows with stride ld: head h at q + row * ld + h / group * dp
  const void* k;
  const void* v;            // head h at v + row * ld + h * vp
  const void* gate;         // rows with stride ldg, heads like v's; null: no output gate
  const float* z;           // [rows, ldz]: gate pre-activations without bias, input gates at [h], forget gates at [f_off + h]
  const float* i_bias;      // [H]
  const float* f_bias;
  const float* norm;        // [H, vp]
  const float* rate;        // STATE_SPACE (which has z and i_bias for the step sizes, and neither f_bias, norm, n nor m): [H]
  const float* skip;        // [H]
  float* S;                 // [slots, H, dp, vp]
  float* n;                 // [slots, H, dp]
  float* m;                 // [slots, H]
  void* out;                // [rows, ldo], head h at h * vp
  long long ld, ldg, ldz, ldo;
  int f_off, H, group, dp, vp, vdim;   // group: heads that share q and k
  float q_scale, cap, eps, out_scale;
};

__device__ __forceinline__ float mem_f32(float v) { return v; }
__device__ __forceinline__ float mem_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void mem_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void mem_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

__device__ __forceinline__ float mem_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float mem_forget_gate(float z, float cap) {
  const float c = cap * tanhf(z / cap);
  return fminf(c, 0.f) - log1pf(expf(-fabsf(c)));
}

// softplus and the decay of a step; decays are often within 1e-3 of one, where an error in the last place of exp would change the
// length of the memory.
__device__ __forceinline__ float state_step(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float state_decay(float rate, float dt) { return 1.f + expm1f(-rate * dt); }

// ---------------------------------------------------------------- token by token
// One block per (item, head).  Thread (r, c): rows r, r + groups, .. of the state and columns 4 c .. 4 c + 3 of each run of
// 4 * lanes columns.  Items are portions (spans) or, with spans null, single rows.  The state of a longer portion is kept
// in shared memory when it fits; with KEEP > 0 a single row's state is asked for ahead of everything else and stays in
// registers, KEEP rows a thread.
constexpr int MS_THREADS = 256;

struct MemoryItems {
  const int* spans;         // [n, 4]: slot, first row, first position, rows; null: row i at pos[i] of slots[i]
  const int* pos;
  const int* slots;
  int in_smem;
};

template <typename T, int RULE, int KEEP>
__global__ void __launch_bounds__(MS_THREADS, KEEP == 8 ? 3 : KEEP == 16 ? 2 : 1)
memory_steps_kernel(const MemoryParams p, const MemoryItems it) {
  extern __shared__ float ms_sm[];
  const int lanes = min(p.vp / 4, MS_THREADS), groups = MS_THREADS / lanes;
  float* s_q = ms_sm;                    // [dp]
  float* s_k = s_q + p.dp;               // [dp]
  float* s_n = s_k + p.dp;               // [dp]
  float* s_v = s_n + p.dp;               // [vp]
  float* s_part = s_v + p.vp;            // [groups, vp]
  float* s_red = s_part + groups * p.vp; // [32]
  float* s_state = s_red + 32;           // [dp, vp] with in_smem
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r = tid / lanes, c = tid - r * lanes;
  int slot, row0, pos0, rows;
  if (it.spans) {
    slot = it.spans[4 * blockIdx.x]; row0 = it.spans[4 * blockIdx.x + 1];
    pos0 = it.spans[4 * blockIdx.x + 2]; rows = it.spans[4 * blockIdx.x + 3];
  } else {
    slot = it.slots[blockIdx.x]; row0 = blockIdx.x; pos0 = it.pos[blockIdx.x]; rows = 1;
  }
  const long long sh = static_cast<long long>(slot) * p.H + h;
  float* S_mem = p.S + sh * p.dp * p.vp;
  float* S = it.in_smem ? s_state : S_mem;
  const long long qk = static_cast<long long>(h / p.group) * p.dp;
  bool fresh = pos0 == 0;
  float4 kept[KEEP > 0 ? KEEP : 1];
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int d = r + i * groups;
      kept[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (r < groups && d < p.dp && !fresh) kept[i] = *reinterpret_cast<const float4*>(S_mem + static_cast<long long>(d) * p.vp + c * 4);
    }
  }
  float m = 0.f;
  if constexpr (RULE == MEMORY) {
    m = fresh ? 0.f : p.m[sh];
    for (int d = tid; d < p.dp; d += MS_THREADS) s_n[d] = fresh ? 0.f : p.n[sh * p.dp + d];
  }
  if (it.in_smem) {
    for (int i = tid * 4; i < p.dp * p.vp; i += MS_THREADS * 4)
      *reinterpret_cast<float4*>(s_state + i) = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(S_mem + i);
    fresh = false;
  }
  const float bi = p.i_bias[h], bf = RULE == MEMORY ? p.f_bias[h] : p.rate[h], skip = RULE == MEMORY ? 0.f : p.skip[h];
  for (int t = 0; t < rows; ++t, fresh = false) {
    const long long row = row0 + t;
    __syncthreads();                     // the state has been loaded; the previous row's vectors have been read
    for (int d = tid; d < p.dp; d += MS_THREADS) {
      s_q[d] = mem_f32(static_cast<const T*>(p.q)[row * p.ld + qk + d]) * p.q_scale;
      s_k[d] = mem_f32(static_cast<const T*>(p.k)[row * p.ld + qk + d]);
    }
    for (int d = tid; d < p.vp; d += MS_THREADS) s_v[d] = mem_f32(static_cast<const T*>(p.v)[row * p.ld + static_cast<long long>(h) * p.vp + d]);
    float keep, add;
    if constexpr (RULE == MEMORY) {
      const float gi = mem_input_gate(p.z[row * p.ldz + h] + bi, p.cap), gf = mem_forget_gate(p.z[row * p.ldz + p.f_off + h] + bf, p.cap);
      const float mm = fmaxf(gf + m, gi);
      keep = expf(gf + m - mm);
      add = expf(gi - mm);
      m = mm;
    } else {
      add = state_step(p.z[row * p.ldz + h] + bi);
      keep = state_decay(bf, add);
    }
    __syncthreads();
    if constexpr (RULE == MEMORY) {
      float dot = 0.f;
      for (int d = tid; d < p.dp; d += MS_THREADS) {
        const float nn = keep * s_n[d] + add * s_k[d];
        s_n[d] = nn;
        dot += nn * s_q[d];
      }
      dot = warp_sum(dot);
      if (lane == 0) s_red[warp] = dot;
    }
    if constexpr (KEEP > 0) {
      if (r < groups) {
        const float4 v4 = *reinterpret_cast<const float4*>(s_v + c * 4);
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < KEEP; ++i) {
          const int d = r + i * groups;
          if (d >= p.dp) continue;
          const float kd = add * s_k[d], qd = s_q[d];
          float4 s = kept[i];
          s.x = keep * s.x + kd * v4.x; s.y = keep * s.y + kd * v4.y;
          s.z = keep * s.z + kd * v4.z; s.w = keep * s.w + kd * v4.w;
          *reinterpret_cast<float4*>(S_mem + static_cast<long long>(d) * p.vp + c * 4) = s;
          acc.x += s.x * qd; acc.y += s.y * qd; acc.z += s.z * qd; acc.w += s.w * qd;
        }
        *reinterpret_cast<float4*>(s_part + r * p.vp + c * 4) = acc;
      }
    } else if (r < groups)
      for (int j = c * 4; j < p.vp; j += lanes * 4) {
        const float4 v4 = *reinterpret_cast<const float4*>(s_v + j);
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int d = r; d < p.dp; d += groups) {
          float4* at = reinterpret_cast<float4*>(S + static_cast<long long>(d) * p.vp + j);
          const float kd = add * s_k[d], qd = s_q[d];
          float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *at;
          s.x = keep * s.x + kd * v4.x; s.y = keep * s.y + kd * v4.y;
          s.z = keep * s.z + kd * v4.z; s.w = keep * s.w + kd * v4.w;
          *at = s;
          acc.x += s.x * qd; acc.y += s.y * qd; acc.z += s.z * qd; acc.w += s.w * qd;
        }
        *reinterpret_cast<float4*>(s_part + r * p.vp + j) = acc;
      }
    __syncthreads();
    if constexpr (RULE == STATE_SPACE) {
      for (int j = tid; j < p.vp; j += MS_THREADS) {
        float o = skip * s_v[j];
        for (int g = 0; g < groups; ++g) o += s_part[g * p.vp + j];
        if (p.gate) {
          const float z = mem_f32(static_cast<const T*>(p.gate)[row * p.ldg + static_cast<long long>(h) * p.vp + j]);
          o *= z / (1.f + expf(-z));
        }
        mem_store(static_cast<T*>(p.out) + row * p.ldo + static_cast<long long>(h) * p.vp + j, o);
      }
      continue;
    }
    float dot = 0.f;
#pragma unroll
    for (int w = 0; w < MS_THREADS / 32; ++w) dot += s_red[w];
    const float inv = 1.f / (fmaxf(fabsf(dot), expf(-m)) + 1e-6f);
    float sum = 0.f;
    for (int j = tid; j < p.vp; j += MS_THREADS) {
      float o = 0.f;
      for (int g = 0; g < groups; ++g) o += s_part[g * p.vp + j];
      o *= inv;
      s_part[j] = o;                     // column j belongs to this thread alone from here on
      sum += o * o;
    }
    sum = warp_sum(sum);
    if (lane == 0) s_red[16 + warp] = sum;
    __syncthreads();
    sum = 0.f;
#pragma unroll
    for (int w = 0; w < MS_THREADS / 32; ++w) sum += s_red[16 + w];
    const float rn = p.out_scale / sqrtf(sum / static_cast<float>(p.vdim) + p.eps);
    for (int j = tid; j < p.vp; j += MS_THREADS) {
      float o = s_part[j] * rn * p.norm[static_cast<long long>(h) * p.vp + j];
      if (p.gate) o *= 1.f / (1.f + expf(-mem_f32(static_cast<const T*>(p.gate)[row * p.ldg + static_cast<long long>(h) * p.vp + j])));
      mem_store(static_cast<T*>(p.out) + row * p.ldo + static_cast<long long>(h) * p.vp + j, o);
    }
  }
  __syncthreads();
  if constexpr (RULE == MEMORY) {
    for (int d = tid; d < p.dp; d += MS_THREADS) p.n[sh * p.dp + d] = s_n[d];
    if (tid == 0) p.m[sh] = m;
  }
  if (it.in_smem)
    for (int i = tid * 4; i < p.dp * p.vp; i += MS_THREADS * 4) *reinterpret_cast<float4*>(S_mem + i) = *reinterpret_cast<const float4*>(s_state + i);
}

// ---------------------------------------------------------------- chunks
constexpr int MC_ROWS = 128;      // tokens of a chunk
constexpr int MC_CHUNK = MC_ROWS * 128;          // bytes of a 64-column tile of 128 rows
constexpr int MC_GATE_WARPS = 32;
constexpr int MC_UPDATE_THREADS = 256;
constexpr int MC_OUT_THREADS = 160;

struct MemoryChunks {
  const int* spans;         // [n_spans, 4]: slot, first row, first position, rows
  const int* span_chunks;   // [n_spans]: first chunk
  const int* chunks;        // [n_chunks, 4]: span, first row, rows, number within the portion
  float* a2;                // [H, ldt] fp32, in powers of two: a_t
  float* x2;                // x_t
  float* floor;             // e^-m_t
  float* start2;            // [n_chunks, H]: M
  float* end2;              // [n_chunks, H]: x of the last token
  float* U;                 // [n_chunks, H, dp, vw]
  float* Un;                // [n_chunks, H, dp]
  __nv_bfloat16* Sb;        // [2, n_chunks, H, dp, vw]: states at the chunks' starts, high and low halves
  float* nb;                // [n_chunks, H, dp]
  long long ldt;
  int n_spans, n_chunks, vw;      // vw: vp rounded up to 64
  int* status;
};

// One block per (head, portion), a warp per chunk, up to MC_GATE_WARPS chunks at a time.
__global__ void __launch_bounds__(MC_GATE_WARPS * 32)
memory_gates_kernel(const MemoryParams p, const MemoryChunks c) {
  __shared__ float s_sum[MC_GATE_WARPS], s_max[MC_GATE_WARPS], s_start[MC_GATE_WARPS];
  __shared__ float s_carry;
  const int h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* span = c.spans + 4 * blockIdx.y;
  const int slot = span[0], row0 = span[1], pos0 = span[2], rows = span[3];
  const int n_chunks = (rows + MC_ROWS - 1) / MC_ROWS, first = c.span_chunks[blockIdx.y];
  float* m_slot = p.m + static_cast<long long>(slot) * p.H + h;
  const float bi = p.i_bias[h], bf = p.f_bias[h];
  if (threadIdx.x == 0) s_carry = pos0 == 0 ? 0.f : *m_slot;
  for (int base = 0; base < n_chunks; base += MC_GATE_WARPS) {
    const int k = base + warp, t0 = k * MC_ROWS + lane * 4;
    float b[4], a[4], x[4];
    float sum = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float f = 0.f;
      a[e] = -INFINITY;
      if (k < n_chunks && t0 + e < rows) {
        const float* z = p.z + (static_cast<long long>(row0) + t0 + e) * p.ldz;
        f = mem_forget_gate(z[p.f_off + h] + bf, p.cap);
        a[e] = mem_input_gate(z[h] + bi, p.cap);
      }
      sum += f;
      b[e] = sum;
    }
    float before = sum;                                // sums of the lanes ahead
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, before, o);
      if (lane >= o) before += v;
    }
    const float total = __shfl_sync(0xffffffffu, before, 31);
    before = __shfl_up_sync(0xffffffffu, before, 1);
    if (lane == 0) before = 0.f;
    float mx = -INFINITY;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      b[e] += before;
      a[e] -= b[e];
      mx = fmaxf(mx, a[e]);
      x[e] = mx;
    }
    float ahead = mx;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, ahead, o);
      if (lane >= o) ahead = fmaxf(ahead, v);
    }
    const float top = __shfl_sync(0xffffffffu, ahead, 31);
    ahead = __shfl_up_sync(0xffffffffu, ahead, 1);
    if (lane == 0) ahead = -INFINITY;
    if (lane == 0) { s_sum[warp] = total; s_max[warp] = top; }
    __syncthreads();
    if (threadIdx.x == 0) {
      float m = s_carry;
      for (int w = 0; w < MC_GATE_WARPS && base + w < n_chunks; ++w) {
        s_start[w] = m;
        m = s_sum[w] + fmaxf(m, s_max[w]);
      }
      s_carry = m;
    }
    __syncthreads();
    if (k < n_chunks) {
      const float start = s_start[warp];
      const long long at = static_cast<long long>(h) * c.ldt + row0 + t0;
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (t0 + e < rows) {
          const float xe = fmaxf(start, fmaxf(ahead, x[e]));
          c.a2[at + e] = a[e] * 1.4426950408889634f;
          c.x2[at + e] = xe * 1.4426950408889634f;
          c.floor[at + e] = expf(-(b[e] + xe));
        }
      if (lane == 0) {
        c.start2[static_cast<long long>(first + k) * p.H + h] = start * 1.4426950408889634f;
        c.end2[static_cast<long long>(first + k) * p.H + h] = fmaxf(start, top) * 1.4426950408889634f;
      }
    }
    __syncthreads();                                   // s_start has been read
  }
  if (threadIdx.x == 0) *m_slot = s_carry;
}

// The same for the state-space rule, where chunks do not wait for one another: a warp per (head, chunk).
__global__ void __launch_bounds__(256)
state_gates_kernel(const MemoryParams p, const MemoryChunks c) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long tasks = static_cast<long long>(c.n_chunks) * p.H;
  for (long long task = static_cast<long long>(blockIdx.x) * 8 + warp; task < tasks; task += static_cast<long long>(gridDim.x) * 8) {
    const int k = static_cast<int>(task / p.H), h = static_cast<int>(task - static_cast<long long>(k) * p.H);
    const int row0 = c.chunks[4 * k + 1], rows = c.chunks[4 * k + 2], t0 = lane * 4;
    const float bias = p.i_bias[h], rate = p.rate[h];
    float dt[4], b[4], sum = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      dt[e] = t0 + e < rows ? state_step(p.z[(static_cast<long long>(row0) + t0 + e) * p.ldz + h] + bias) : 0.f;
      sum -= rate * dt[e];
      b[e] = sum;
    }
    float before = sum;                                // sums of the lanes ahead
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, before, o);
      if (lane >= o) before += v;
    }
    const float total = __shfl_sync(0xffffffffu, before, 31);
    before = __shfl_up_sync(0xffffffffu, before, 1);
    if (lane == 0) before = 0.f;
    const long long at = static_cast<long long>(h) * c.ldt + row0 + t0;
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (t0 + e < rows) {
        const float b2 = (b[e] + before) * 1.4426950408889634f;
        c.a2[at + e] = log2f(dt[e]) - b2;              // a step of zero: -inf, a weight of zero
        c.x2[at + e] = -b2;
      }
    if (lane == 0) {
      c.start2[task] = 0.f;
      c.end2[task] = -total * 1.4426950408889634f;
    }
  }
}

// 16-byte unit `unit` of row `row` in a tile of 64-column pieces with 128-byte swizzle.
__device__ __forceinline__ uint32_t mc_unit(int row, int unit) {
  return static_cast<uint32_t>(unit >> 3) * MC_CHUNK + static_cast<uint32_t>(row) * 128u + (static_cast<uint32_t>((unit & 7) ^ (row & 7)) << 4);
}

// U of one (chunk, head).  MEMORY: the keys' tile [128 tokens, 128] is weighted in place (its low halves go to a second tile) and
// multiplied as the transposed A operand with V; their weighted sum is the normaliser's contribution.  STATE_SPACE: V, which is
// narrower, is weighted instead.
template <int VC, int RULE>
struct MemUpdate {       // shared memory: K | low halves of what is weighted | V
  static constexpr int LO = RULE == MEMORY ? 2 : VC, OFF_LO = 2 * MC_CHUNK, OFF_V = OFF_LO + LO * MC_CHUNK, OFF_N = OFF_V + VC * MC_CHUNK,
                       OFF_W = OFF_N + (RULE == MEMORY ? 16 * 128 * 4 : 0), OFF_BAR = OFF_W + MC_ROWS * 4, SMEM = OFF_BAR + 64 + 1024;
};

template <int VC, int RULE>
__global__ void __launch_bounds__(MC_UPDATE_THREADS)
memory_update_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const MemoryParams p, const MemoryChunks c) {
  using Cfg = MemUpdate<VC, RULE>;
  constexpr int OFF_LO = Cfg::OFF_LO, OFF_V = Cfg::OFF_V, OFF_N = Cfg::OFF_N, OFF_W = Cfg::OFF_W, OFF_BAR = Cfg::OFF_BAR;
  constexpr uint32_t COLS = VC == 1 ? 64 : (VC == 2 ? 128 : 256);
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const uint32_t sbase = smem_u32(smem);
  float* s_n = reinterpret_cast<float*>(smem + OFF_N);             // [16][128]
  float* s_w = reinterpret_cast<float*>(smem + OFF_W);
  const uint32_t bar_k = sbase + OFF_BAR, bar_v = bar_k + 8, bar_m = bar_k + 16;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + OFF_BAR + 24);
  volatile int* abort_word = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
  const int h = blockIdx.y;
  const int* ch = c.chunks + 4 * blockIdx.x;
  const int row0 = ch[1], rows = ch[2];
  const long long ph = static_cast<long long>(blockIdx.x) * p.H + h;
  if (tid == 0) {
    *abort_word = 0;
    mbar_init(bar_k, 1);
    mbar_init(bar_v, 1);
    mbar_init(bar_m, 1);
    fence_mbar_init();
  }
  if (warp == 0) {
    tmem_alloc(smem_u32(tmem_slot), COLS);
    tmem_relinquish();
  }
  const float end2 = c.end2[ph];
  if (tid < MC_ROWS) s_w[tid] = tid < rows ? exp2f(c.a2[static_cast<long long>(h) * c.ldt + row0 + tid] - end2) : 0.f;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  if (tid == 0) {
    mbar_expect_tx(bar_k, 2 * MC_CHUNK);
    for (int i = 0; i < 2; ++i) tma_load_2d(sbase + i * MC_CHUNK, &tmK, bar_k, h / p.group * p.dp + i * 64, row0);
    mbar_expect_tx(bar_v, VC * MC_CHUNK);
    for (int i = 0; i < VC; ++i) tma_load_2d(sbase + OFF_V + i * MC_CHUNK, &tmV, bar_v, h * p.vp + i * 64, row0);
  }
  bool ok = mbar_wait(RULE == MEMORY ? bar_k : bar_v, 0, abort_word, FT_ERR_TIMEOUT_EPILOGUE);
  if (ok) {
    constexpr int UNITS = RULE == MEMORY ? 16 : 8 * VC, STEP = MC_UPDATE_THREADS / UNITS, OFF_IN = RULE == MEMORY ? 0 : OFF_V;
    const int unit = tid % UNITS, r0 = tid / UNITS;
    float acc[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.f;
#pragma unroll
    for (int i = 0; i < (MC_ROWS + STEP - 1) / STEP; ++i) {
      const int row = r0 + STEP * i;
      if (r0 >= STEP || row >= MC_ROWS) continue;
      uint4* at = reinterpret_cast<uint4*>(smem + OFF_IN + mc_unit(row, unit));
      const float w = s_w[row];
      float f[8], hi[8];
      unpack8(*at, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        f[e] *= w;
        if constexpr (RULE == MEMORY) acc[e] += f[e];
      }
      const uint4 packed = pack8(f);
      unpack8(packed, hi);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] -= hi[e];
      *at = packed;
      *reinterpret_cast<uint4*>(smem + OFF_LO + mc_unit(row, unit)) = pack8(f);
    }
    if constexpr (RULE == MEMORY) {
#pragma unroll
      for (int e = 0; e < 8; ++e) s_n[r0 * 128 + unit * 8 + e] = acc[e];
    }
  }
  fence_proxy_async_smem();
  __syncthreads();
  if (tid == 0 && ok && mbar_wait(RULE == MEMORY ? bar_v : bar_k, 0, abort_word, FT_ERR_TIMEOUT_MMA)) {
    constexpr int OFF_A = RULE == MEMORY ? OFF_LO : 0, OFF_B = RULE == MEMORY ? 0 : OFF_LO - OFF_V;      // from the high to the low halves
    if (RULE == STATE_SPACE) tc_fence_after();
    constexpr uint32_t idesc = make_idesc_f16(128, VC * 64, 1, 1, 1);
#pragma unroll
    for (int half = 0; half < 2; ++half)
#pragma unroll
      for (int kk = 0; kk < MC_ROWS / 16; ++kk)
        umma_f16_ss(tmem, make_smem_desc_sw128(sbase + half * OFF_A + kk * 2048, MC_CHUNK, 1024),
                    make_smem_desc_sw128(sbase + OFF_V + half * OFF_B + kk * 2048, MC_CHUNK, 1024), idesc, (half > 0 || kk > 0) ? 1u : 0u);
    umma_commit(bar_m);
  }
  if (RULE == MEMORY && tid < p.dp && ok) {
    float n = 0.f;
#pragma unroll
    for (int g = 0; g < 16; ++g) n += s_n[g * 128 + tid];
    c.Un[ph * p.dp + tid] = n;
  }
  ok = mbar_wait(bar_m, 0, abort_word, FT_ERR_TIMEOUT_EPILOGUE) && ok;
  ok = __all_sync(0xffffffffu, ok);
  if (ok) {
    tc_fence_after();
    const int ew = warp & 3, d = ew * 32 + lane;
    if (ew * 32 < p.dp) {                              // whole warps: the TMEM load is a warp-wide instruction
      float* dst = c.U + (ph * p.dp + d) * c.vw;
      for (int col = (warp >> 2) * 32; col < VC * 64; col += 64) {
        uint32_t t[32];
        tmem_ld_32x32(tmem + (static_cast<uint32_t>(ew * 32) << 16) + col, t);
        tmem_ld_wait();
        if (d < p.dp) {
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            float f[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(t[g * 8 + e]);
            store8_sector(dst + col + g * 8, f);
          }
        }
      }
    }
  } else if (tid == 0) {                               // let copies in flight land before the block leaves
    const unsigned long long t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, COLS);
  }
  if (tid == 0 && *abort_word != 0 && c.status) atomicCAS(c.status, 0, *abort_word);
}

// The states of a portion's chunks, one after another: a thread owns four elements of S (and the first block one of n).
constexpr int MC_AHEAD = 4;       // contributions loaded together
template <int RULE>
__global__ void __launch_bounds__(256)
memory_carry_kernel(const MemoryParams p, const MemoryChunks c) {
  const int h = blockIdx.y;
  const int* span = c.spans + 4 * blockIdx.z;
  const int slot = span[0], pos0 = span[2], rows = span[3];
  const int n_chunks = (rows + MC_ROWS - 1) / MC_ROWS, first = c.span_chunks[blockIdx.z];
  const long long sh = static_cast<long long>(slot) * p.H + h;
  const int i = (blockIdx.x * 256 + threadIdx.x) * 4;
  const long long per = static_cast<long long>(p.dp) * c.vw, low = static_cast<long long>(c.n_chunks) * p.H * per;
  auto factor = [&](int k) {
    const long long at = static_cast<long long>(first + k) * p.H + h;
    return exp2f(c.start2[at] - c.end2[at]);
  };
  if (i < p.dp * c.vw) {
    const int d = i / c.vw, col = i - d * c.vw;
    float4* S = reinterpret_cast<float4*>(p.S + (sh * p.dp + d) * p.vp + col);
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    if (col < p.vp && pos0 > 0) s = *S;
    for (int k0 = 0; k0 < n_chunks; k0 += MC_AHEAD) {
      float4 u[MC_AHEAD];
      float g[MC_AHEAD];
#pragma unroll
      for (int j = 0; j < MC_AHEAD; ++j)
        if (k0 + j < n_chunks) {
          u[j] = __ldcs(reinterpret_cast<const float4*>(c.U + (static_cast<long long>(first + k0 + j) * p.H + h) * per + i));
          g[j] = factor(k0 + j);
        }
#pragma unroll
      for (int j = 0; j < MC_AHEAD; ++j)
        if (k0 + j < n_chunks) {
          __nv_bfloat16* at = c.Sb + (static_cast<long long>(first + k0 + j) * p.H + h) * per + i;
          const uint32_t h0 = pack_bf16x2(s.x, s.y), h1 = pack_bf16x2(s.z, s.w);
          const float2 f0 = unpack_bf16x2(h0), f1 = unpack_bf16x2(h1);
          *reinterpret_cast<uint2*>(at) = make_uint2(h0, h1);
          *reinterpret_cast<uint2*>(at + low) = make_uint2(pack_bf16x2(s.x - f0.x, s.y - f0.y), pack_bf16x2(s.z - f1.x, s.w - f1.y));
          s.x = g[j] * s.x + u[j].x; s.y = g[j] * s.y + u[j].y; s.z = g[j] * s.z + u[j].z; s.w = g[j] * s.w + u[j].w;
        }
    }
    if (col < p.vp) *S = s;
  }
  if (RULE == MEMORY && blockIdx.x == 0 && static_cast<int>(threadIdx.x) < p.dp) {
    float n = pos0 > 0 ? p.n[sh * p.dp + threadIdx.x] : 0.f;
    for (int k = 0; k < n_chunks; ++k) {
      const long long at = (static_cast<long long>(first + k) * p.H + h) * p.dp + threadIdx.x;
      c.nb[at] = n;
      n = factor(k) * n + c.Un[at];
    }
    p.n[sh * p.dp + threadIdx.x] = n;
  }
}

// Outputs of one (chunk, head).  Warps 0-3: thread = token.  Warp 4: copies and products.  Shared memory: Q | K, then the low half
// of the state | the high half of the state, then V; at the end the gate lies over Q (and what follows), and the results over it.
// With APART the state's high half has a place of its own, so that V is loaded at once, and the gate as soon as that half has been
// read, to whose place it and then the results go.
template <int DC, int VC, int RULE>
struct MemOut {
  static constexpr int MID = DC > VC ? DC : VC;
  static constexpr bool APART = RULE == STATE_SPACE && VC <= 2;
  static constexpr int OFF_K = DC * MC_CHUNK, OFF_V = OFF_K + MID * MC_CHUNK, OFF_H = APART ? OFF_V + VC * MC_CHUNK : OFF_V,
                       OFF_G = APART ? OFF_H : 0, OFF_A = OFF_H + VC * MC_CHUNK, OFF_NB = OFF_A + MC_ROWS * 4,
                       OFF_W = OFF_NB + 128 * 4, OFF_BAR = OFF_W + VC * 64 * 4, SMEM = OFF_BAR + 128 + 1024;
  static constexpr uint32_t COLS = VC <= 2 ? 256 : 512, COL_LOW = 64, COL_O = 128;      // scores (then P high | low), outputs
};

template <int DC, int VC, int RULE>
__global__ void __launch_bounds__(MC_OUT_THREADS)
memory_output_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                     const __grid_constant__ CUtensorMap tmS, const __grid_constant__ CUtensorMap tmG, const MemoryParams p,
                     const MemoryChunks c) {
  using Cfg = MemOut<DC, VC, RULE>;
  constexpr bool APART = Cfg::APART;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const uint32_t sQ = smem_u32(smem), sK = sQ + Cfg::OFF_K, sV = sQ + Cfg::OFF_V, sH = sQ + Cfg::OFF_H;
  float* s_a = reinterpret_cast<float*>(smem + Cfg::OFF_A);
  float* s_nb = reinterpret_cast<float*>(smem + Cfg::OFF_NB);
  float* s_w = reinterpret_cast<float*>(smem + Cfg::OFF_W);
  enum { QK = 0, HIGH, LOW, V, SCORE, HIGH_DONE, INTER, Q_READ, P_FULL, GATE, OUT, NBARS };
  auto bar = [&](int i) { return sQ + Cfg::OFF_BAR + 8u * i; };
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + Cfg::OFF_BAR + 8 * NBARS);
  volatile int* abort_word = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
  const int h = blockIdx.y;
  const int* ch = c.chunks + 4 * blockIdx.x;
  const int row0 = ch[1], rows = ch[2];
  const bool fresh = ch[3] == 0 && c.spans[4 * ch[0] + 2] == 0;                 // nothing ahead of this chunk
  const long long ph = static_cast<long long>(blockIdx.x) * p.H + h, gate_at = static_cast<long long>(h) * c.ldt + row0;
  if (tid == 0) {
    *abort_word = 0;
    for (int i = 0; i < NBARS; ++i) mbar_init(bar(i), i == P_FULL || i == Q_READ ? 4 : 1);
    fence_mbar_init();
  }
  if (warp == 4) {
    tmem_alloc(smem_u32(tmem_slot), Cfg::COLS);
    tmem_relinquish();
  }
  if (tid < MC_ROWS) s_a[tid] = tid < rows ? c.a2[gate_at + tid] : -INFINITY;
  if (RULE == MEMORY && tid < p.dp) s_nb[tid] = fresh ? 0.f : c.nb[ph * p.dp + tid];
  if (RULE == MEMORY) for (int i = tid; i < p.vp; i += MC_OUT_THREADS) s_w[i] = p.norm[static_cast<long long>(h) * p.vp + i];
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;

  if (warp == 4) {
    if (lane == 0) {
      auto wait = [&](int i) { return mbar_wait(bar(i), 0, abort_word, FT_ERR_TIMEOUT_MMA); };
      auto load_v = [&]() {
        mbar_expect_tx(bar(V), VC * MC_CHUNK);
        for (int i = 0; i < VC; ++i) tma_load_2d(sV + i * MC_CHUNK, &tmV, bar(V), h * p.vp + i * 64, row0);
      };
      auto load_state = [&](int b, uint32_t dst, long long row) {
        mbar_expect_tx(bar(b), static_cast<uint32_t>(p.dp) * 128u * VC);
        for (int i = 0; i < VC; ++i) tma_load_2d(dst + i * MC_CHUNK, &tmS, bar(b), i * 64, static_cast<int>(row));
      };
      constexpr uint32_t idesc_score = make_idesc_f16(128, 128, 1, 0, 0), idesc_out = make_idesc_f16(128, VC * 64, 1, 0, 1);
      auto q_state = [&](uint32_t state, bool first) {                          // O (+)= Q times one half of the state
        for (int kk = 0; kk < p.dp / 16; ++kk)
          umma_f16_ss(tmem + Cfg::COL_O, make_smem_desc_sw128(sQ + (kk >> 2) * MC_CHUNK + (kk & 3) * 32, 16, 1024),
                      make_smem_desc_sw128(state + kk * 2048, MC_CHUNK, 1024), idesc_out, (first && kk == 0) ? 0u : 1u);
      };
      mbar_expect_tx(bar(QK), 2 * DC * MC_CHUNK);
      for (int i = 0; i < DC; ++i) {
        tma_load_2d(sQ + i * MC_CHUNK, &tmQ, bar(QK), h / p.group * p.dp + i * 64, row0);
        tma_load_2d(sK + i * MC_CHUNK, &tmK, bar(QK), h / p.group * p.dp + i * 64, row0);
      }
      auto load_gate = [&]() {
        mbar_expect_tx(bar(GATE), VC * MC_CHUNK);
        for (int i = 0; i < VC; ++i) tma_load_2d(sQ + Cfg::OFF_G + i * MC_CHUNK, &tmG, bar(GATE), h * p.vp + i * 64, row0);
      };
      if (!fresh) load_state(HIGH, sH, ph * p.dp);
      if (fresh || APART) load_v();
      if (fresh && APART && p.gate) load_gate();
      bool ok = wait(QK);
      if (ok) {
        tc_fence_after();
        for (int kk = 0; kk < p.dp / 16; ++kk) {
          const uint32_t off = (kk >> 2) * MC_CHUNK + (kk & 3) * 32;
          umma_f16_ss(tmem, make_smem_desc_sw128(sQ + off, 16, 1024), make_smem_desc_sw128(sK + off, 16, 1024), idesc_score, kk > 0 ? 1u : 0u);
        }
        umma_commit(bar(SCORE));
      }
      if (!fresh) {
        if (ok && (ok = wait(HIGH))) {
          tc_fence_after();
          q_state(sH, true);
          umma_commit(bar(HIGH_DONE));
        }
        if (ok && (ok = wait(SCORE))) load_state(LOW, sK, (static_cast<long long>(c.n_chunks) * p.H + ph) * p.dp);    // K has been read
        if (ok && (ok = wait(HIGH_DONE))) {
          if (!APART) load_v();
          else if (p.gate) load_gate();
        }
        if (ok && (ok = wait(LOW))) {
          tc_fence_after();
          q_state(sK, false);
          umma_commit(bar(INTER));
        }
      }
      // the last product with Q has finished and every token has read its own: the gate takes the place
      if (!APART && ok && p.gate && (ok = wait(fresh ? SCORE : INTER)) && (ok = wait(Q_READ))) load_gate();
      if (ok && (ok = wait(V)) && (ok = wait(P_FULL))) {
        tc_fence_after();
#pragma unroll
        for (int half = 0; half < 2; ++half)
#pragma unroll
          for (int kk = 0; kk < MC_ROWS / 16; ++kk)
            umma_f16_ts(tmem + Cfg::COL_O, tmem + half * Cfg::COL_LOW + kk * 8, make_smem_desc_sw128(sV + kk * 2048, MC_CHUNK, 1024), idesc_out,
                        (fresh && half == 0 && kk == 0) ? 0u : 1u);
        umma_commit(bar(OUT));
      }
      if (!ok) {                                       // let copies in flight land before the block leaves
        const unsigned long long t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
      }
    }
  } else {
    const bool row_ok = tid < rows;
    const float x2 = row_ok ? c.x2[gate_at + tid] : 0.f, floor_m = RULE == MEMORY && row_ok ? c.floor[gate_at + tid] : 1.f;
    const float skip = RULE == STATE_SPACE ? p.skip[h] : 0.f;
    const float inter = (fresh || !row_ok) ? 0.f : exp2f(c.start2[ph] - x2) * p.q_scale;
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(warp * 32) << 16);
    float den = 0.f;
    auto wait = [&](int i) { return __all_sync(0xffffffffu, mbar_wait(bar(i), 0, abort_word, FT_ERR_TIMEOUT_EPILOGUE)); };
    bool ok = wait(QK);
    if (RULE == MEMORY && ok && !fresh) {              // q times the normaliser at the chunk's start
      for (int u = 0; u < p.dp / 8; ++u) {
        float f[8];
        unpack8(*reinterpret_cast<const uint4*>(smem + mc_unit(tid, u)), f);
#pragma unroll
        for (int e = 0; e < 8; ++e) den += f[e] * s_nb[u * 8 + e];
      }
      den *= inter;
    }
    __syncwarp();
    if (ok && lane == 0) mbar_arrive(bar(Q_READ));
    ok = ok && wait(SCORE);
    if (ok) {
      tc_fence_after();
      uint32_t lows[2][16];                            // low halves of the first two groups wait until their scores' place is free
#pragma unroll
      for (int j = 0; j < 4; ++j) {                    // 32 keys at a time; the high halves of a group lie over scores already read
        uint32_t hi[16], lo[16];
        if (j <= warp) {
          uint32_t t[32];
          tmem_ld_32x32(lane_addr + j * 32, t);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            float v[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const int key = j * 32 + 2 * i + e;
              const float w = fast_exp2(s_a[key] - x2);
              v[e] = key <= tid ? __uint_as_float(t[2 * i + e]) * p.q_scale * w : 0.f;
              if constexpr (RULE == MEMORY) den += v[e];
            }
            hi[i] = pack_bf16x2(v[0], v[1]);
            const float2 r = unpack_bf16x2(hi[i]);
            lo[i] = pack_bf16x2(v[0] - r.x, v[1] - r.y);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 16; ++i) hi[i] = lo[i] = 0u;
        }
        tmem_st_32x16(lane_addr + j * 16, hi);
        if (j < 2) {
#pragma unroll
          for (int i = 0; i < 16; ++i) lows[j][i] = lo[i];
        } else if (j == 2) {
          tmem_st_32x16(lane_addr + Cfg::COL_LOW, lows[0]);          // scores 64 .. 95 have been read
          tmem_st_32x16(lane_addr + Cfg::COL_LOW + 16, lows[1]);
#pragma unroll
          for (int i = 0; i < 16; ++i) lows[0][i] = lo[i];
        } else {
          tmem_st_32x16(lane_addr + Cfg::COL_LOW + 32, lows[0]);
          tmem_st_32x16(lane_addr + Cfg::COL_LOW + 48, lo);
        }
      }
      if (!fresh) {
        ok = wait(INTER);
        if (ok) {
          tc_fence_after();
#pragma unroll 1
          for (int col = 0; col < VC * 64; col += 32) {
            uint32_t t[32];
            tmem_ld_32x32(lane_addr + Cfg::COL_O + col, t);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 32; ++e) t[e] = __float_as_uint(__uint_as_float(t[e]) * inter);
            tmem_st_32x32(lane_addr + Cfg::COL_O + col, t);
          }
        }
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (ok && lane == 0) mbar_arrive(bar(P_FULL));
    }
    if (ok) ok = wait(OUT);
    if (ok) {
      tc_fence_after();
      float r = 1.f;
      if constexpr (RULE == MEMORY) {
        const float inv = 1.f / (fmaxf(fabsf(den), floor_m) + 1e-6f);
        float sum = 0.f;
#pragma unroll
        for (int col = 0; col < VC * 64; col += 32) {
          uint32_t t[32];
          tmem_ld_32x32(lane_addr + Cfg::COL_O + col, t);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 32; ++e) {
            const float o = __uint_as_float(t[e]) * inv;
            if (col + e < p.vp) sum += o * o;
          }
        }
        r = p.out_scale * inv / sqrtf(sum / static_cast<float>(p.vdim) + p.eps);
      }
      if (p.gate) ok = wait(GATE);
#pragma unroll 1
      for (int col = 0; col < VC * 64; col += 32) {
        if (col >= p.vp) break;
        uint32_t t[32];
        tmem_ld_32x32(lane_addr + Cfg::COL_O + col, t);
        tmem_ld_wait();
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          uint4* at = reinterpret_cast<uint4*>(smem + Cfg::OFF_G + mc_unit(tid, col / 8 + g));
          float f[8], z[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = RULE == MEMORY ? __uint_as_float(t[g * 8 + e]) * r * s_w[col + g * 8 + e] : __uint_as_float(t[g * 8 + e]);
          if constexpr (RULE == STATE_SPACE) {
            unpack8(*reinterpret_cast<const uint4*>(smem + Cfg::OFF_V + mc_unit(tid, col / 8 + g)), z);
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] += skip * z[e];
          }
          if (p.gate) {
            unpack8(*at, z);
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] = __fdividef(RULE == MEMORY ? f[e] : f[e] * z[e], 1.f + __expf(-z[e]));
          }
          *at = pack8(f);
        }
      }
      __syncwarp();
      // the warp's rows, contiguous pieces of a row by neighbouring lanes
      const int units = p.vp / 8, live = min(32, rows - warp * 32) * units;
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + (static_cast<long long>(row0) + warp * 32) * p.ldo + static_cast<long long>(h) * p.vp;
      for (int i = lane; ok && i < live; i += 32) {
        const int rr = i / units, u = i - rr * units;
        *reinterpret_cast<uint4*>(out + rr * p.ldo + u * 8) = *reinterpret_cast<const uint4*>(smem + Cfg::OFF_G + mc_unit(warp * 32 + rr, u));
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 4) {
    tc_fence_after();
    tmem_dealloc(tmem, Cfg::COLS);
  }
  if (tid == 0 && *abort_word != 0 && c.status) atomicCAS(c.status, 0, *abort_word);
}

static bool mem_aligned(std::initializer_list<const void*> ps) {
  uintptr_t v = 0;
  for (const void* p : ps) v |= reinterpret_cast<uintptr_t>(p);
  return (v & 15) == 0;
}

static int memory_params(MemoryParams& p, const void* q, const void* k, const void* v, long long ld, const void* gate, long long ldg, const float* z,
                         long long ldz, const float* i_bias, float* S, void* out, long long ldo, int H, int group, int dp, int vp) {
  FT_REQUIRE(q && k && v && z && i_bias && S && out, "matrix memory: null pointer");
  FT_REQUIRE(H > 0 && H < 65536 && group > 0 && H % group == 0 && dp > 0 && dp % 16 == 0 && vp > 0 && vp % 16 == 0 && ld % 8 == 0 && ldo % 8 == 0 &&
                 ldg % 8 == 0 && (!gate || ldg >= static_cast<long long>(H) * vp) && ldo >= static_cast<long long>(H) * vp && ldz >= H,
             "matrix memory: %d heads of %d x %d in groups of %d", H, dp, vp, group);
  FT_REQUIRE(mem_aligned({q, k, v, gate, S, out}), "matrix memory: pointers must be 16-byte aligned");
  p = MemoryParams{};
  p.q = q; p.k = k; p.v = v; p.gate = gate; p.z = z; p.i_bias = i_bias; p.S = S; p.out = out;
  p.ld = ld; p.ldg = ldg; p.ldz = ldz; p.ldo = ldo; p.H = H; p.group = group; p.dp = dp; p.vp = vp; p.vdim = vp;
  p.q_scale = 1.f; p.out_scale = 1.f; p.cap = 1.f;
  return FT_E_OK;
}

// What the memory rule has beside the common operands.
static int memory_gates(MemoryParams& p, int f_off, const float* f_bias, const float* norm, float* n, float* m, int vdim, float q_scale, float cap,
                        float eps, float out_scale) {
  FT_REQUIRE(f_bias && norm && n && m && vdim > 0 && vdim <= p.vp && f_off >= p.H && p.ldz >= f_off + p.H && cap > 0.f, "matrix memory: gates or null pointer");
  FT_REQUIRE(mem_aligned({n, norm}), "matrix memory: pointers must be 16-byte aligned");
  p.f_off = f_off; p.f_bias = f_bias; p.norm = norm; p.n = n; p.m = m; p.vdim = vdim;
  p.q_scale = q_scale; p.cap = cap; p.eps = eps; p.out_scale = out_scale;
  return FT_E_OK;
}

static int state_rates(MemoryParams& p, const float* rate, const float* skip) {
  FT_REQUIRE(rate && skip, "state space: null pointer");
  p.rate = rate; p.skip = skip;
  return FT_E_OK;
}

template <int RULE>
static int run_steps(const MemoryParams& p, const int* spans, const int* pos, const int* slots, int n_items, int f32, cudaStream_t stream) {
  FT_REQUIRE(spans || (pos && slots), "matrix memory: neither portions nor rows");
  if (n_items <= 0) return FT_E_OK;
  MemoryItems it = {spans, pos, slots, 0};
  const int lanes = p.vp / 4 < MS_THREADS ? p.vp / 4 : MS_THREADS, groups = MS_THREADS / lanes;
  size_t smem = sizeof(float) * (3 * static_cast<size_t>(p.dp) + p.vp + static_cast<size_t>(groups) * p.vp + 32);
  const size_t state = sizeof(float) * static_cast<size_t>(p.dp) * p.vp;
  if (spans && smem + state <= 200 * 1024) {
    it.in_smem = 1;
    smem += state;
  }
  FT_REQUIRE(smem <= 200 * 1024, "matrix memory: heads of %d x %d are too large", p.dp, p.vp);
  const dim3 grid(n_items, p.H);
  const int per_thread = !spans && p.vp <= 4 * MS_THREADS ? (p.dp + groups - 1) / groups : 1 << 30;     // rows of the state
  auto kern = f32 ? memory_steps_kernel<float, RULE, 0> : memory_steps_kernel<__nv_bfloat16, RULE, 0>;
  if (!f32 && per_thread <= 8) kern = memory_steps_kernel<__nv_bfloat16, RULE, 8>;
  else if (!f32 && per_thread <= 16) kern = memory_steps_kernel<__nv_bfloat16, RULE, 16>;
  FT_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  kern<<<grid, MS_THREADS, smem, stream>>>(p, it);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

}  // namespace ft

using namespace ft;

// The recurrence token by token over n_items portions (spans int32 [n_items, 4]) or, with spans null, over rows 0 .. n_items
// - 1 that are their sequences' only token (pos, slots).  Operands as in MemoryParams, bf16 or fp32 with f32; head sizes dp and
// vp multiples of 16, of whose values vdim exist (padding is zero).
FT_API int ft_memory_steps(const void* q, const void* k, const void* v, const void* gate, long long ld, const float* z, long long ldz,
                           int f_off, const float* i_bias, const float* f_bias, const float* norm, float* S, float* n, float* m,
                           void* out, long long ldo, int H, int dp, int vp, int vdim, float q_scale, float cap, float eps,
                           float out_scale, const int* spans, const int* pos, const int* slots, int n_items, int f32, int device,
                           cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  MemoryParams p;
  if (int rc = memory_params(p, q, k, v, ld, gate, ld, z, ldz, i_bias, S, out, ldo, H, 1, dp, vp)) return rc;
  if (int rc = memory_gates(p, f_off, f_bias, norm, n, m, vdim, q_scale, cap, eps, out_scale)) return rc;
  return run_steps<MEMORY>(p, spans, pos, slots, n_items, f32, stream);
}

// The state-space rule token by token: v (x) [rows, H * vp], k and q (B and C) [rows, H / group * dp] with row stride ld, gate [rows, ldg] or
// null, z fp32 [rows, ldz] (step sizes ahead of bias and softplus), bias, rate and skip fp32 [H], S fp32 [slots, H, dp, vp].  Items as in
// ft_memory_steps.
FT_API int ft_state_steps(const void* q, const void* k, const void* v, long long ld, const void* gate, long long ldg, const float* z, long long ldz,
                          const float* bias, const float* rate, const float* skip, float* S, void* out, long long ldo, int H, int group, int dp,
                          int vp, const int* spans, const int* pos, const int* slots, int n_items, int f32, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  MemoryParams p;
  if (int rc = memory_params(p, q, k, v, ld, gate, ldg, z, ldz, bias, S, out, ldo, H, group, dp, vp)) return rc;
  if (int rc = state_rates(p, rate, skip)) return rc;
  return run_steps<STATE_SPACE>(p, spans, pos, slots, n_items, f32, stream);
}

// Whole portions of bf16 rows in chunks (see the top of this file): dp up to 128, vp up to 256.  rows: rows of the packed
// projection.  spans [n_spans, 4] and chunks [n_chunks, 4] (span, first row, rows up to 128, number within the portion;
// portion after portion) int32, span_chunks [n_spans]: first chunk of a portion.  scratch: ft_memory_scratch bytes.
static long long memory_scratch_at(int rows, int H, int dp, int vp, int n_chunks, long long* at) {
  const long long vw = (vp + 63) / 64 * 64, ldt = (rows + 31) / 32 * 32, ch = static_cast<long long>(n_chunks) * H;
  const long long sizes[9] = {H * ldt * 4, H * ldt * 4, H * ldt * 4, ch * 4, ch * 4, ch * dp * vw * 4, ch * dp * 4, ch * dp * vw * 4, ch * dp * 4};
  long long total = 0;
  for (int i = 0; i < 9; ++i) {
    if (at) at[i] = total;
    total += (sizes[i] + 255) / 256 * 256;
  }
  return total;
}

FT_API long long ft_memory_scratch(int rows, int H, int dp, int vp, int n_chunks) { return memory_scratch_at(rows, H, dp, vp, n_chunks, nullptr); }

template <int DC, int VC, int RULE>
static int launch_memory(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const CUtensorMap& ts, const CUtensorMap& tg,
                         const MemoryParams& p, const MemoryChunks& c, int device, cudaStream_t stream) {
  constexpr int UPDATE_SMEM = MemUpdate<VC, RULE>::SMEM;
  constexpr int OUT_SMEM = MemOut<DC, VC, RULE>::SMEM;
  auto update = memory_update_kernel<VC, RULE>;
  auto output = memory_output_kernel<DC, VC, RULE>;
  static bool attr_set[64] = {false};
  if (!attr_set[device]) {
    FT_CUDA_CHECK(cudaFuncSetAttribute(update, cudaFuncAttributeMaxDynamicSharedMemorySize, UPDATE_SMEM));
    FT_CUDA_CHECK(cudaFuncSetAttribute(output, cudaFuncAttributeMaxDynamicSharedMemorySize, OUT_SMEM));
    attr_set[device] = true;
  }
  if (RULE == MEMORY) {
    memory_gates_kernel<<<dim3(p.H, c.n_spans), MC_GATE_WARPS * 32, 0, stream>>>(p, c);
  } else {
    const long long blocks = (static_cast<long long>(c.n_chunks) * p.H + 7) / 8, cap = sm_count(device) * 16;
    state_gates_kernel<<<static_cast<int>(blocks < cap ? blocks : cap), 256, 0, stream>>>(p, c);
  }
  FT_CUDA_CHECK(cudaGetLastError());
  update<<<dim3(c.n_chunks, p.H), MC_UPDATE_THREADS, UPDATE_SMEM, stream>>>(tk, tv, p, c);
  FT_CUDA_CHECK(cudaGetLastError());
  memory_carry_kernel<RULE><<<dim3((p.dp * c.vw / 4 + 255) / 256, p.H, c.n_spans), 256, 0, stream>>>(p, c);
  FT_CUDA_CHECK(cudaGetLastError());
  output<<<dim3(c.n_chunks, p.H), MC_OUT_THREADS, OUT_SMEM, stream>>>(tq, tk, tv, ts, tg, p, c);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch(4);
  return FT_E_OK;
}

template <int RULE>
static int run_chunks(const MemoryParams& p, int rows, const int* spans, int n_spans, const int* span_chunks, const int* chunks, int n_chunks,
                      void* scratch, int device, cudaStream_t stream) {
  const int H = p.H, dp = p.dp, vp = p.vp;
  FT_REQUIRE(dp <= 128 && vp <= 256, "matrix memory: heads of %d x %d are too large for chunks", dp, vp);
  FT_REQUIRE(rows > 0 && spans && span_chunks && chunks && scratch && (reinterpret_cast<uintptr_t>(scratch) & 255) == 0, "matrix memory: null pointer or unaligned scratch");
  if (n_spans <= 0 || n_chunks <= 0) return FT_E_OK;
  FT_REQUIRE(n_spans < 65536 && 2ll * n_chunks * H * dp < (1ll << 31), "matrix memory: too many portions or chunks");
  long long at[9];
  memory_scratch_at(rows, H, dp, vp, n_chunks, at);
  char* base = static_cast<char*>(scratch);
  MemoryChunks c;
  c.spans = spans; c.span_chunks = span_chunks; c.chunks = chunks;
  c.a2 = reinterpret_cast<float*>(base + at[0]); c.x2 = reinterpret_cast<float*>(base + at[1]); c.floor = reinterpret_cast<float*>(base + at[2]);
  c.start2 = reinterpret_cast<float*>(base + at[3]); c.end2 = reinterpret_cast<float*>(base + at[4]); c.U = reinterpret_cast<float*>(base + at[5]);
  c.Un = reinterpret_cast<float*>(base + at[6]); c.Sb = reinterpret_cast<__nv_bfloat16*>(base + at[7]); c.nb = reinterpret_cast<float*>(base + at[8]);
  c.ldt = (rows + 31) / 32 * 32; c.n_spans = n_spans; c.n_chunks = n_chunks; c.vw = (vp + 63) / 64 * 64;
  c.status = device_status_word(device);
  CUtensorMap tq, tk, tv, ts, tg;
  const uint64_t stride = static_cast<uint64_t>(p.ld) * 2, keys = static_cast<uint64_t>(H / p.group) * dp;
  if (int rc = make_tmap_2d(&tq, p.q, 2, keys, rows, stride, 64, MC_ROWS, 3)) return rc;
  if (int rc = make_tmap_2d(&tk, p.k, 2, keys, rows, stride, 64, MC_ROWS, 3)) return rc;
  if (int rc = make_tmap_2d(&tv, p.v, 2, static_cast<uint64_t>(H) * vp, rows, stride, 64, MC_ROWS, 3)) return rc;
  if (int rc = make_tmap_2d(&tg, p.gate ? p.gate : p.v, 2, static_cast<uint64_t>(H) * vp, rows, p.gate ? static_cast<uint64_t>(p.ldg) * 2 : stride, 64, MC_ROWS, 3)) return rc;
  if (int rc = make_tmap_2d(&ts, c.Sb, 2, c.vw, 2 * static_cast<uint64_t>(n_chunks) * H * dp, static_cast<uint64_t>(c.vw) * 2, 64, dp, 3)) return rc;
#define FT_MC(DCN)                                                              \
  switch (c.vw / 64) {                                                          \
    case 1: return launch_memory<DCN, 1, RULE>(tq, tk, tv, ts, tg, p, c, device, stream); \
    case 2: return launch_memory<DCN, 2, RULE>(tq, tk, tv, ts, tg, p, c, device, stream); \
    case 3: return launch_memory<DCN, 3, RULE>(tq, tk, tv, ts, tg, p, c, device, stream); \
    default: return launch_memory<DCN, 4, RULE>(tq, tk, tv, ts, tg, p, c, device, stream); \
  }
  if (dp <= 64) { FT_MC(1) }
  FT_MC(2)
#undef FT_MC
}

FT_API int ft_memory_chunks(const void* q, const void* k, const void* v, const void* gate, long long ld, const float* z, long long ldz,
                            int f_off, const float* i_bias, const float* f_bias, const float* norm, float* S, float* n, float* m,
                            void* out, long long ldo, int H, int dp, int vp, int vdim, float q_scale, float cap, float eps,
                            float out_scale, int rows, const int* spans, int n_spans, const int* span_chunks, const int* chunks,
                            int n_chunks, void* scratch, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  MemoryParams p;
  if (int rc = memory_params(p, q, k, v, ld, gate, ld, z, ldz, i_bias, S, out, ldo, H, 1, dp, vp)) return rc;
  if (int rc = memory_gates(p, f_off, f_bias, norm, n, m, vdim, q_scale, cap, eps, out_scale)) return rc;
  return run_chunks<MEMORY>(p, rows, spans, n_spans, span_chunks, chunks, n_chunks, scratch, device, stream);
}

// The state-space rule over whole portions of bf16 rows in chunks: operands as in ft_state_steps, portions and chunks as in
// ft_memory_chunks, scratch of ft_state_scratch bytes.
FT_API long long ft_state_scratch(int rows, int H, int dp, int vp, int n_chunks) { return memory_scratch_at(rows, H, dp, vp, n_chunks, nullptr); }

FT_API int ft_state_chunks(const void* q, const void* k, const void* v, long long ld, const void* gate, long long ldg, const float* z, long long ldz,
                           const float* bias, const float* rate, const float* skip, float* S, void* out, long long ldo, int H, int group, int dp,
                           int vp, int rows, const int* spans, int n_spans, const int* span_chunks, const int* chunks, int n_chunks, void* scratch,
                           int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  MemoryParams p;
  if (int rc = memory_params(p, q, k, v, ld, gate, ldg, z, ldz, bias, S, out, ldo, H, group, dp, vp)) return rc;
  if (int rc = state_rates(p, rate, skip)) return rc;
  return run_chunks<STATE_SPACE>(p, rows, spans, n_spans, span_chunks, chunks, n_chunks, scratch, device, stream);
}
