// Matrix memories (the recurrence of xLSTM's mLSTM): per head a state S [dim, vdim] and a normaliser n [dim], both relative
// to a running maximum m of the logarithmic gates,
//
//   i = cap tanh((zi + bi) / cap),  f = logsigmoid(cap tanh((zf + bf) / cap))
//   m' = max(f + m, i),  S' = e^(f + m - m') S + e^(i - m') k v^T,  n' likewise with k alone
//   o = S'^T q / (max(|n'.q|, e^-m') + 1e-6)
//
// followed by an RMS norm of every head's o, a weight, the sigmoid of an output gate and a constant factor.  Gates, states
// and all arithmetic of the recurrence are fp32; q, k, v and the output gate come from a packed projection.
//
//   ft_memory_steps   token by token: rows that are their sequence's only token, short portions, any sizes, bf16 or fp32
//
// A slot needs no clearing: what a sequence has seen follows from its positions, and position 0 starts from zero.
#include <initializer_list>

#include "row_vec.cuh"

namespace ft {

struct MemoryParams {
  const void* q;            // rows of a packed projection with stride ld: head h at q + row * ld + h * dp
  const void* k;
  const void* v;            // head h at v + row * ld + h * vp
  const void* gate;         // like v; null: no output gate
  const float* z;           // [rows, ldz]: gate pre-activations without bias, input gates at [h], forget gates at [f_off + h]
  const float* i_bias;      // [H]
  const float* f_bias;
  const float* norm;        // [H, vp]
  float* S;                 // [slots, H, dp, vp]
  float* n;                 // [slots, H, dp]
  float* m;                 // [slots, H]
  void* out;                // [rows, ldo], head h at h * vp
  long long ld, ldz, ldo;
  int f_off, H, dp, vp, vdim;
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

// ---------------------------------------------------------------- token by token
// One block per (item, head).  Thread (r, c): rows r, r + groups, .. of the state and columns 4 c .. 4 c + 3 of each run of
// 4 * lanes columns.  Items are portions (spans) or, with spans null, single rows.  The state of a longer portion is kept
// in shared memory when it fits.
constexpr int MS_THREADS = 256;

struct MemoryItems {
  const int* spans;         // [n, 4]: slot, first row, first position, rows; null: row i at pos[i] of slots[i]
  const int* pos;
  const int* slots;
  int in_smem;
};

template <typename T>
__global__ void __launch_bounds__(MS_THREADS)
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
  bool fresh = pos0 == 0;
  float m = fresh ? 0.f : p.m[sh];
  for (int d = tid; d < p.dp; d += MS_THREADS) s_n[d] = fresh ? 0.f : p.n[sh * p.dp + d];
  if (it.in_smem) {
    for (int i = tid * 4; i < p.dp * p.vp; i += MS_THREADS * 4)
      *reinterpret_cast<float4*>(s_state + i) = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(S_mem + i);
    fresh = false;
  }
  const float bi = p.i_bias[h], bf = p.f_bias[h];
  for (int t = 0; t < rows; ++t, fresh = false) {
    const long long row = row0 + t;
    __syncthreads();                     // the state has been loaded; the previous row's vectors have been read
    for (int d = tid; d < p.dp; d += MS_THREADS) {
      s_q[d] = mem_f32(static_cast<const T*>(p.q)[row * p.ld + static_cast<long long>(h) * p.dp + d]) * p.q_scale;
      s_k[d] = mem_f32(static_cast<const T*>(p.k)[row * p.ld + static_cast<long long>(h) * p.dp + d]);
    }
    for (int d = tid; d < p.vp; d += MS_THREADS) s_v[d] = mem_f32(static_cast<const T*>(p.v)[row * p.ld + static_cast<long long>(h) * p.vp + d]);
    const float gi = mem_input_gate(p.z[row * p.ldz + h] + bi, p.cap), gf = mem_forget_gate(p.z[row * p.ldz + p.f_off + h] + bf, p.cap);
    const float mm = fmaxf(gf + m, gi);
    const float keep = expf(gf + m - mm), add = expf(gi - mm);
    m = mm;
    __syncthreads();
    float dot = 0.f;
    for (int d = tid; d < p.dp; d += MS_THREADS) {
      const float nn = keep * s_n[d] + add * s_k[d];
      s_n[d] = nn;
      dot += nn * s_q[d];
    }
    dot = warp_sum(dot);
    if (lane == 0) s_red[warp] = dot;
    if (r < groups)
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
    dot = 0.f;
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
      if (p.gate) o *= 1.f / (1.f + expf(-mem_f32(static_cast<const T*>(p.gate)[row * p.ld + static_cast<long long>(h) * p.vp + j])));
      mem_store(static_cast<T*>(p.out) + row * p.ldo + static_cast<long long>(h) * p.vp + j, o);
    }
  }
  __syncthreads();
  for (int d = tid; d < p.dp; d += MS_THREADS) p.n[sh * p.dp + d] = s_n[d];
  if (tid == 0) p.m[sh] = m;
  if (it.in_smem)
    for (int i = tid * 4; i < p.dp * p.vp; i += MS_THREADS * 4) *reinterpret_cast<float4*>(S_mem + i) = *reinterpret_cast<const float4*>(s_state + i);
}

static bool mem_aligned(std::initializer_list<const void*> ps) {
  uintptr_t v = 0;
  for (const void* p : ps) v |= reinterpret_cast<uintptr_t>(p);
  return (v & 15) == 0;
}

static int memory_params(MemoryParams& p, const void* q, const void* k, const void* v, const void* gate, long long ld, const float* z,
                         long long ldz, int f_off, const float* i_bias, const float* f_bias, const float* norm, float* S, float* n,
                         float* m, void* out, long long ldo, int H, int dp, int vp, int vdim, float q_scale, float cap, float eps,
                         float out_scale) {
  FT_REQUIRE(q && k && v && z && i_bias && f_bias && norm && S && n && m && out, "matrix memory: null pointer");
  FT_REQUIRE(H > 0 && H < 65536 && dp > 0 && dp % 16 == 0 && vp > 0 && vp % 16 == 0 && vdim > 0 && vdim <= vp && ld % 8 == 0 && ldo % 8 == 0 &&
                 ldo >= static_cast<long long>(H) * vp && f_off >= H && ldz >= f_off + H && cap > 0.f,
             "matrix memory: %d heads of %d x %d", H, dp, vp);
  FT_REQUIRE(mem_aligned({q, k, v, gate, S, n, out, norm}), "matrix memory: pointers must be 16-byte aligned");
  p.q = q; p.k = k; p.v = v; p.gate = gate; p.z = z; p.i_bias = i_bias; p.f_bias = f_bias; p.norm = norm; p.S = S; p.n = n; p.m = m;
  p.out = out; p.ld = ld; p.ldz = ldz; p.ldo = ldo; p.f_off = f_off; p.H = H; p.dp = dp; p.vp = vp; p.vdim = vdim;
  p.q_scale = q_scale; p.cap = cap; p.eps = eps; p.out_scale = out_scale;
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
  if (int rc = memory_params(p, q, k, v, gate, ld, z, ldz, f_off, i_bias, f_bias, norm, S, n, m, out, ldo, H, dp, vp, vdim, q_scale, cap, eps, out_scale))
    return rc;
  FT_REQUIRE(spans || (pos && slots), "ft_memory_steps: neither portions nor rows");
  if (n_items <= 0) return FT_E_OK;
  MemoryItems it = {spans, pos, slots, 0};
  const int lanes = vp / 4 < MS_THREADS ? vp / 4 : MS_THREADS, groups = MS_THREADS / lanes;
  size_t smem = sizeof(float) * (3 * static_cast<size_t>(dp) + vp + static_cast<size_t>(groups) * vp + 32);
  const size_t state = sizeof(float) * static_cast<size_t>(dp) * vp;
  if (spans && smem + state <= 200 * 1024) {
    it.in_smem = 1;
    smem += state;
  }
  FT_REQUIRE(smem <= 200 * 1024, "ft_memory_steps: heads of %d x %d are too large", dp, vp);
  const dim3 grid(n_items, H);
  auto kern = f32 ? memory_steps_kernel<float> : memory_steps_kernel<__nv_bfloat16>;
  FT_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  kern<<<grid, MS_THREADS, smem, stream>>>(p, it);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}
