// Memory-bound transformer kernels for sm_100a: RMSNorm (+ fused residual add)
// forward/backward, rotary embedding (both pair conventions) forward/backward,
// SwiGLU forward/backward, embedding gather / scatter-add, dynamic tanh on an fp32
// residual stream (optionally fused with the embedding gather), and the step between a
// decoder layer's packed input projection and its attention (projection norms, query
// temperature, KV append, MLP activation).
//
// Semantics follow the reference: RMSNorm = x * rsqrt(mean(x^2) + eps) * w with fp32
// statistics (ferrotorch-gpu/src/bf16.rs:1340-1346, kernels.rs:10578, 10725); RoPE
// rotates the pair (d, d + D/2) ("half" / HF convention, bf16.rs:1850-1855) or
// (2d, 2d+1) (interleaved, ferrotorch-nn/src/transformer.rs:66-72) with the backward
// of transformer.rs:132-156; SwiGLU = silu(gate) * up (ferrotorch-llama/src/gpu.rs:696-703).
// Unlike the reference (one launch per op, 256-thread 1-D grids) every kernel moves
// 16-byte vectors, keeps the row in registers between the statistics pass and the
// scale pass, and fuses the neighbouring residual add / gate multiply.
#include "row_vec.cuh"

namespace ft {

constexpr int NORM_THREADS = 256;
constexpr int NORM_MAX_VEC = 4;  // 4 vec * 8 elems * 256 thr = rows up to 8192 wide in registers

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = (threadIdx.x < (blockDim.x >> 5)) ? red[threadIdx.x] : 0.f;
  if (w == 0) {
    t = warp_sum(t);
    if (l == 0) red[0] = t;
  }
  __syncthreads();
  return red[0];
}
__device__ __forceinline__ float block_max(float v, float* red) {
  v = warp_max(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = (threadIdx.x < (blockDim.x >> 5)) ? red[threadIdx.x] : -INFINITY;
  if (w == 0) {
    t = warp_max(t);
    if (l == 0) red[0] = t;
  }
  __syncthreads();
  return red[0];
}


// ---------------------------------------------------------------- RMSNorm forward
// y = (x [+ delta]) * rstd * w ; if delta != null also writes res_out = x + delta.
// One block per row, grid-stride over rows. H % 8 == 0.
__global__ void __launch_bounds__(NORM_THREADS)
rmsnorm_fwd_kernel(const __nv_bfloat16* __restrict__ x, const __nv_bfloat16* __restrict__ delta,
                   const __nv_bfloat16* __restrict__ w, __nv_bfloat16* __restrict__ y,
                   __nv_bfloat16* __restrict__ res_out, float* __restrict__ rstd_out, int rows, int H,
                   float eps) {
  __shared__ float red[32];
  const int nvec = H >> 3;
  for (int row = blockIdx.x; row < rows; row += gridDim.x) {
    const uint4* xr = reinterpret_cast<const uint4*>(x + static_cast<size_t>(row) * H);
    const uint4* dr = delta ? reinterpret_cast<const uint4*>(delta + static_cast<size_t>(row) * H) : nullptr;
    float vals[NORM_MAX_VEC][8];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NORM_MAX_VEC; ++i) {
      const int v = threadIdx.x + i * NORM_THREADS;
      if (v < nvec) {
        unpack8(xr[v], vals[i]);
        if (dr) {
          float d[8];
          unpack8(dr[v], d);
#pragma unroll
          for (int j = 0; j < 8; ++j) vals[i][j] += d[j];
          if (res_out) {
            // round the residual stream to bf16 once; the statistics use the rounded value
            uint4 packed = pack8(vals[i]);
            reinterpret_cast<uint4*>(res_out + static_cast<size_t>(row) * H)[v] = packed;
            unpack8(packed, vals[i]);
          }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += vals[i][j] * vals[i][j];
      }
    }
    const float tot = block_sum(ss, red);
    const float rstd = rsqrtf(tot / static_cast<float>(H) + eps);
    if (threadIdx.x == 0 && rstd_out) rstd_out[row] = rstd;
#pragma unroll
    for (int i = 0; i < NORM_MAX_VEC; ++i) {
      const int v = threadIdx.x + i * NORM_THREADS;
      if (v < nvec) {
        float wv[8], o[8];
        unpack8(reinterpret_cast<const uint4*>(w)[v], wv);
#pragma unroll
        for (int j = 0; j < 8; ++j) o[j] = vals[i][j] * rstd * wv[j];
        reinterpret_cast<uint4*>(y + static_cast<size_t>(row) * H)[v] = pack8(o);
      }
    }
  }
}

// ---------------------------------------------------------------- RMSNorm backward
// dx = rstd * (g - xhat * mean(g * xhat)) [+ dres], g = dy * w, xhat = x * rstd.
// dw partial sums: each block keeps its columns' sums in registers over the rows it
// owns and writes one fp32 row of the scratch [gridDim.x, H]; rmsnorm_dw_reduce sums it.
__global__ void __launch_bounds__(NORM_THREADS)
rmsnorm_bwd_kernel(const __nv_bfloat16* __restrict__ dy, const __nv_bfloat16* __restrict__ x,
                   const __nv_bfloat16* __restrict__ w, const float* __restrict__ rstd_in,
                   const __nv_bfloat16* __restrict__ dres, __nv_bfloat16* __restrict__ dx,
                   float* __restrict__ dw_partial, int rows, int H) {
  __shared__ float red[32];
  const int nvec = H >> 3;
  float dwacc[NORM_MAX_VEC][8];
#pragma unroll
  for (int i = 0; i < NORM_MAX_VEC; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j) dwacc[i][j] = 0.f;

  for (int row = blockIdx.x; row < rows; row += gridDim.x) {
    const size_t off = static_cast<size_t>(row) * H;
    const float rstd = rstd_in[row];
    float g[NORM_MAX_VEC][8], xh[NORM_MAX_VEC][8];
    float dot = 0.f;
#pragma unroll
    for (int i = 0; i < NORM_MAX_VEC; ++i) {
      const int v = threadIdx.x + i * NORM_THREADS;
      if (v < nvec) {
        float dyv[8], wv[8];
        unpack8(reinterpret_cast<const uint4*>(dy + off)[v], dyv);
        unpack8(reinterpret_cast<const uint4*>(x + off)[v], xh[i]);
        unpack8(reinterpret_cast<const uint4*>(w)[v], wv);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          xh[i][j] *= rstd;
          g[i][j] = dyv[j] * wv[j];
          dot += g[i][j] * xh[i][j];
          dwacc[i][j] += dyv[j] * xh[i][j];
        }
      }
    }
    const float mean_dot = block_sum(dot, red) / static_cast<float>(H);
#pragma unroll
    for (int i = 0; i < NORM_MAX_VEC; ++i) {
      const int v = threadIdx.x + i * NORM_THREADS;
      if (v < nvec) {
        float o[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) o[j] = rstd * (g[i][j] - xh[i][j] * mean_dot);
        if (dres) {
          float r[8];
          unpack8(reinterpret_cast<const uint4*>(dres + off)[v], r);
#pragma unroll
          for (int j = 0; j < 8; ++j) o[j] += r[j];
        }
        reinterpret_cast<uint4*>(dx + off)[v] = pack8(o);
      }
    }
  }
  if (dw_partial) {
    float* out = dw_partial + static_cast<size_t>(blockIdx.x) * H;
#pragma unroll
    for (int i = 0; i < NORM_MAX_VEC; ++i) {
      const int v = threadIdx.x + i * NORM_THREADS;
      if (v < nvec) {
        reinterpret_cast<float4*>(out)[2 * v] = make_float4(dwacc[i][0], dwacc[i][1], dwacc[i][2], dwacc[i][3]);
        reinterpret_cast<float4*>(out)[2 * v + 1] = make_float4(dwacc[i][4], dwacc[i][5], dwacc[i][6], dwacc[i][7]);
      }
    }
  }
}

// dw[h] (+)= sum_b partial[b, h]; writes bf16 or fp32.  A block owns 32 columns (one 128-byte
// segment of every partial row); its 8 warps each walk every 8th row with four loads in flight and
// the 8 sub-sums are added in warp order, so the result does not depend on scheduling.
constexpr int DW_RED_COLS = 32, DW_RED_WARPS = 8;
__global__ void __launch_bounds__(DW_RED_COLS * DW_RED_WARPS)
rmsnorm_dw_reduce_kernel(const float* __restrict__ partial, void* __restrict__ dw, int nblocks, int H,
                         int out_f32, int accumulate) {
  __shared__ float sub[DW_RED_WARPS][DW_RED_COLS];
  const int tx = threadIdx.x & (DW_RED_COLS - 1), ty = threadIdx.x / DW_RED_COLS;
  const int h = blockIdx.x * DW_RED_COLS + tx;
  float s0 = 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
  if (h < H) {
    const float* col = partial + h;
    int b = ty;
    for (; b + 3 * DW_RED_WARPS < nblocks; b += 4 * DW_RED_WARPS) {
      s0 += col[static_cast<size_t>(b) * H];
      s1 += col[static_cast<size_t>(b + DW_RED_WARPS) * H];
      s2 += col[static_cast<size_t>(b + 2 * DW_RED_WARPS) * H];
      s3 += col[static_cast<size_t>(b + 3 * DW_RED_WARPS) * H];
    }
    for (; b < nblocks; b += DW_RED_WARPS) s0 += col[static_cast<size_t>(b) * H];
  }
  sub[ty][tx] = (s0 + s1) + (s2 + s3);
  __syncthreads();
  if (ty != 0 || h >= H) return;
  float s = 0.f;
#pragma unroll
  for (int k = 0; k < DW_RED_WARPS; ++k) s += sub[k][tx];
  if (out_f32) {
    float* o = static_cast<float*>(dw);
    o[h] = accumulate ? o[h] + s : s;
  } else {
    __nv_bfloat16* o = static_cast<__nv_bfloat16*>(dw);
    o[h] = __float2bfloat16(accumulate ? __bfloat162float(o[h]) + s : s);
  }
}

// ---------------------------------------------------------------- RoPE
// x: [T, n_heads_total, D] with row stride `ld` (elements) between tokens; rotates
// heads [0, n_rot_heads).  cos/sin: fp32 [max_pos, D/2].  pos: int32 [T] or null
// (then position = (t % seq_len) + pos_offset).  sign = +1 forward, -1 backward.
__global__ void rope_kernel(__nv_bfloat16* __restrict__ x, const float* __restrict__ cos_t,
                            const float* __restrict__ sin_t, const int* __restrict__ pos, int T,
                            int n_rot_heads, int D, long long ld, int seq_len, int pos_offset,
                            int interleaved, float sign) {
  const int half = D >> 1;
  const int pairs_per_tok = n_rot_heads * half;
  const long long total = static_cast<long long>(T) * (pairs_per_tok >> 1);  // 2 pairs / thread
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int t = static_cast<int>(i / (pairs_per_tok >> 1));
    const int r = static_cast<int>(i - static_cast<long long>(t) * (pairs_per_tok >> 1)) * 2;
    const int h = r / half, d = r - h * half;  // d even
    const int p = pos ? pos[t] : (t % seq_len) + pos_offset;
    const float2 c = *reinterpret_cast<const float2*>(cos_t + static_cast<size_t>(p) * half + d);
    float2 s = *reinterpret_cast<const float2*>(sin_t + static_cast<size_t>(p) * half + d);
    s.x *= sign; s.y *= sign;
    __nv_bfloat16* base = x + static_cast<size_t>(t) * ld + static_cast<size_t>(h) * D;
    if (!interleaved) {
      __nv_bfloat162* p1 = reinterpret_cast<__nv_bfloat162*>(base + d);
      __nv_bfloat162* p2 = reinterpret_cast<__nv_bfloat162*>(base + d + half);
      const float2 a = __bfloat1622float2(*p1), b = __bfloat1622float2(*p2);
      *p1 = __floats2bfloat162_rn(a.x * c.x - b.x * s.x, a.y * c.y - b.y * s.y);
      *p2 = __floats2bfloat162_rn(b.x * c.x + a.x * s.x, b.y * c.y + a.y * s.y);
    } else {
      uint2* pp = reinterpret_cast<uint2*>(base + 2 * d);
      uint2 u = *pp;
      const float2 e0 = unpack_bf16x2(u.x), e1 = unpack_bf16x2(u.y);  // (x0,x1), (x2,x3)
      u.x = pack_bf16x2(e0.x * c.x - e0.y * s.x, e0.y * c.x + e0.x * s.x);
      u.y = pack_bf16x2(e1.x * c.y - e1.y * s.y, e1.y * c.y + e1.x * s.y);
      *pp = u;
    }
  }
}

// Vector version: one thread rotates 8 pairs.  Half-rotation layout: 16 bytes from the first
// half of a head and the 16 bytes that pair with them in the second half; interleaved layout:
// 32 contiguous bytes.  cos/sin come as two float4 each.  Needs D % 16 == 0 and 16-byte
// aligned rows (checked by the launcher).
__global__ void rope_vec_kernel(__nv_bfloat16* __restrict__ x, const float* __restrict__ cos_t,
                                const float* __restrict__ sin_t, const int* __restrict__ pos, int T,
                                int n_rot_heads, int D, long long ld, int seq_len, int pos_offset,
                                int interleaved, float sign) {
  const int half = D >> 1;
  const int groups_per_head = half >> 3;                       // 8 pairs per group
  const int groups_per_tok = n_rot_heads * groups_per_head;
  const long long total = static_cast<long long>(T) * groups_per_tok;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int t = static_cast<int>(i / groups_per_tok);
    const int r = static_cast<int>(i - static_cast<long long>(t) * groups_per_tok);
    const int h = r / groups_per_head, d = (r - h * groups_per_head) << 3;   // first pair index
    const int p = pos ? pos[t] : (t % seq_len) + pos_offset;
    const float4* cp = reinterpret_cast<const float4*>(cos_t + static_cast<size_t>(p) * half + d);
    const float4* sp = reinterpret_cast<const float4*>(sin_t + static_cast<size_t>(p) * half + d);
    const float4 c0 = cp[0], c1 = cp[1], s0 = sp[0], s1 = sp[1];
    const float c[8] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w};
    const float sn[8] = {s0.x * sign, s0.y * sign, s0.z * sign, s0.w * sign,
                         s1.x * sign, s1.y * sign, s1.z * sign, s1.w * sign};
    __nv_bfloat16* base = x + static_cast<size_t>(t) * ld + static_cast<size_t>(h) * D;
    float a[8], b[8], oa[8], ob[8];
    if (!interleaved) {
      uint4* p1 = reinterpret_cast<uint4*>(base + d);
      uint4* p2 = reinterpret_cast<uint4*>(base + d + half);
      unpack8(*p1, a);
      unpack8(*p2, b);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        oa[j] = a[j] * c[j] - b[j] * sn[j];
        ob[j] = b[j] * c[j] + a[j] * sn[j];
      }
      *p1 = pack8(oa);
      *p2 = pack8(ob);
    } else {
      uint4* pp = reinterpret_cast<uint4*>(base + 2 * d);
      unpack8(pp[0], a);      // pairs 0..3 as (even, odd)
      unpack8(pp[1], b);      // pairs 4..7
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        oa[2 * j] = a[2 * j] * c[j] - a[2 * j + 1] * sn[j];
        oa[2 * j + 1] = a[2 * j + 1] * c[j] + a[2 * j] * sn[j];
        ob[2 * j] = b[2 * j] * c[4 + j] - b[2 * j + 1] * sn[4 + j];
        ob[2 * j + 1] = b[2 * j + 1] * c[4 + j] + b[2 * j] * sn[4 + j];
      }
      pp[0] = pack8(oa);
      pp[1] = pack8(ob);
    }
  }
}

// ---------------------------------------------------------------- SwiGLU
// gu: [T, 2F] (gate = [:, :F], up = [:, F:]), out: [T, F].  act: 0 silu, 1 relu, 2 gelu(tanh).
__device__ __forceinline__ float act_fwd(float g, int act) {
  if (act == 0) return g / (1.f + __expf(-g));
  if (act == 1) return fmaxf(g, 0.f);
  const float k = 0.7978845608028654f * (g + 0.044715f * g * g * g);
  return 0.5f * g * (1.f + tanhf(k));
}
__device__ __forceinline__ float act_bwd(float g, int act) {
  if (act == 0) {
    const float s = 1.f / (1.f + __expf(-g));
    return s * (1.f + g * (1.f - s));
  }
  if (act == 1) return g > 0.f ? 1.f : 0.f;
  const float k = 0.7978845608028654f * (g + 0.044715f * g * g * g);
  const float t = tanhf(k);
  return 0.5f * (1.f + t) + 0.5f * g * (1.f - t * t) * 0.7978845608028654f * (1.f + 3.f * 0.044715f * g * g);
}
// Two vectors per thread with all loads issued first and streaming (evict-first) hints on the
// inputs, which are read exactly once.
__global__ void swiglu_fwd2_kernel(const __nv_bfloat16* __restrict__ gu, __nv_bfloat16* __restrict__ out,
                                   long long T, int F, long long ld_gu, int act) {
  const int fv = F >> 3;
  const long long total = T * fv;
  const long long stride = static_cast<long long>(gridDim.x) * blockDim.x;
  for (long long i0 = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i0 < total; i0 += 2 * stride) {
    const long long i1 = i0 + stride < total ? i0 + stride : i0;
    const long long t0 = i0 / fv, t1 = i1 / fv;
    const int v0 = static_cast<int>(i0 - t0 * fv), v1 = static_cast<int>(i1 - t1 * fv);
    const uint4* r0 = reinterpret_cast<const uint4*>(gu + t0 * ld_gu);
    const uint4* r1 = reinterpret_cast<const uint4*>(gu + t1 * ld_gu);
    const uint4 g0 = __ldcs(r0 + v0), u0 = __ldcs(r0 + fv + v0), g1 = __ldcs(r1 + v1), u1 = __ldcs(r1 + fv + v1);
    float g[8], u[8], o[8];
    unpack8(g0, g);
    unpack8(u0, u);
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = act_fwd(g[j], act) * u[j];
    reinterpret_cast<uint4*>(out + t0 * F)[v0] = pack8(o);
    if (i1 != i0) {
      unpack8(g1, g);
      unpack8(u1, u);
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] = act_fwd(g[j], act) * u[j];
      reinterpret_cast<uint4*>(out + t1 * F)[v1] = pack8(o);
    }
  }
}
__global__ void swiglu_bwd2_kernel(const __nv_bfloat16* __restrict__ dy, const __nv_bfloat16* __restrict__ gu,
                                   __nv_bfloat16* __restrict__ dgu, long long T, int F, long long ld_gu,
                                   int act) {
  const int fv = F >> 3;
  const long long total = T * fv;
  const long long stride = static_cast<long long>(gridDim.x) * blockDim.x;
  for (long long i0 = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i0 < total; i0 += 2 * stride) {
    const long long i1 = i0 + stride < total ? i0 + stride : i0;
    const long long tt[2] = {i0 / fv, i1 / fv};
    const int vv[2] = {static_cast<int>(i0 - tt[0] * fv), static_cast<int>(i1 - tt[1] * fv)};
    uint4 gq[2], uq[2], dq[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const uint4* row = reinterpret_cast<const uint4*>(gu + tt[k] * ld_gu);
      gq[k] = __ldcs(row + vv[k]);
      uq[k] = __ldcs(row + fv + vv[k]);
      dq[k] = __ldcs(reinterpret_cast<const uint4*>(dy + tt[k] * F) + vv[k]);
    }
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      if (k == 1 && i1 == i0) break;
      float g[8], u[8], d[8], dg[8], du[8];
      unpack8(gq[k], g);
      unpack8(uq[k], u);
      unpack8(dq[k], d);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        dg[j] = d[j] * u[j] * act_bwd(g[j], act);
        du[j] = d[j] * act_fwd(g[j], act);
      }
      uint4* orow = reinterpret_cast<uint4*>(dgu + tt[k] * ld_gu);
      orow[vv[k]] = pack8(dg);
      orow[fv + vv[k]] = pack8(du);
    }
  }
}

// ---------------------------------------------------------------- embedding
__global__ void embedding_fwd_kernel(const long long* __restrict__ ids, const __nv_bfloat16* __restrict__ w,
                                     __nv_bfloat16* __restrict__ out, int T, int H, int vocab) {
  const int hv = H >> 3;
  for (int t = blockIdx.x; t < T; t += gridDim.x) {
    long long id = ids[t];
    if (id < 0 || id >= vocab) id = 0;  // host validates; never read out of range
    const uint4* src = reinterpret_cast<const uint4*>(w + static_cast<size_t>(id) * H);
    uint4* dst = reinterpret_cast<uint4*>(out + static_cast<size_t>(t) * H);
    for (int v = threadIdx.x; v < hv; v += blockDim.x) dst[v] = src[v];
  }
}
__global__ void embedding_bwd_kernel(const long long* __restrict__ ids, const __nv_bfloat16* __restrict__ dy,
                                     __nv_bfloat16* __restrict__ dw, int T, int H, int vocab) {
  const int h2 = H >> 1;
  for (int t = blockIdx.x; t < T; t += gridDim.x) {
    const long long id = ids[t];
    if (id < 0 || id >= vocab) continue;
    const __nv_bfloat162* src = reinterpret_cast<const __nv_bfloat162*>(dy + static_cast<size_t>(t) * H);
    __nv_bfloat162* dst = reinterpret_cast<__nv_bfloat162*>(dw + static_cast<size_t>(id) * H);
    for (int v = threadIdx.x; v < h2; v += blockDim.x) atomicAdd(dst + v, src[v]);
  }
}

// ---------------------------------------------------------------- dynamic tanh
// y = (tanh(alpha * x) * w + b) * scale, element by element (no row statistic), fp32 input and
// parameters.  With `ids` the input row is table[ids[row]] (a row of the embedding, TI) and is also
// written to x_out, the fp32 residual stream.  A thread owns eight columns and walks rows, so w and b
// stay in registers.
template <typename TI, typename TO>
__global__ void __launch_bounds__(NORM_THREADS)
dyt_kernel(const TI* __restrict__ x, const long long* __restrict__ ids, int vocab, float* __restrict__ x_out,
           const float* __restrict__ alpha_p, const float* __restrict__ w, const float* __restrict__ b,
           TO* __restrict__ y, int rows, int H, long long ldx, long long ldy, float scale) {
  const int v = blockIdx.x * blockDim.x + threadIdx.x;
  if (v >= (H >> 3)) return;
  const float alpha = *alpha_p;
  float wv[8], bv[8];
  load8(w + v * 8, wv);
  load8(b + v * 8, bv);
  for (int row = blockIdx.y; row < rows; row += gridDim.y) {
    long long src = row;
    if (ids) {
      src = ids[row];
      if (src < 0 || src >= vocab) src = 0;  // host validates; never read out of range
    }
    float f[8], o[8];
    load8(x + src * ldx + v * 8, f);
    if (x_out) store8(x_out + static_cast<long long>(row) * H + v * 8, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = (tanhf(alpha * f[j]) * wv[j] + bv[j]) * scale;
    store8(y + static_cast<long long>(row) * ldy + v * 8, o);
  }
}

// The activation ahead of a bf16 store: 0.5 (1 + tanh u) = 1 / (1 + exp(-2 u)) needs one exponential and one
// approximate division, where tanhf makes the kernel compute-bound.  fp32 rows keep act_fwd.
__device__ __forceinline__ float act_row(float g, int act, const __nv_bfloat16*) {
  if (act != 2) return act_fwd(g, act);
  return g * __fdividef(1.f, 1.f + __expf(-1.5957691216057308f * (g + 0.044715f * g * g * g)));
}
__device__ __forceinline__ float act_row(float g, int act, const float*) { return act_fwd(g, act); }

// ---------------------------------------------------------------- packed projection -> attention
// One pass over a row of the packed input projection [ .. q .. k .. v .. up .. ] of a decoder layer
// whose attention and feed-forward read the same input:
//   q   RMS-normalised over the whole projection (all heads at once), times the query temperature
//       1 + coef * ln(floor((pos + 1) / every) + 1), written back in place
//   k   RMS-normalised over the whole projection, written to its cache page
//   v   copied to its cache page
//   up  act(up), written to the input of the output projection
// Each part is optional (null weight: no norm; coef 0: no temperature; no act output: no MLP).  The
// means divide by q_count / k_count, the true sizes of the projections: padded elements are zero.
struct QkvFinishParams {
  void* packed;                 // [rows, ld]
  long long ld;
  const int* pos;
  const int* slots;
  const int* block_table;
  void* k_cache;
  void* v_cache;
  const float* q_weight;
  const float* k_weight;
  void* act_out;                // [rows, ld_act]
  long long ld_act;
  int rows, q_off, q_n, k_off, k_n, v_off, v_n, up_off, up_n, q_count, k_count;
  float eps, temp_coef;
  double temp_every;
  int act, block_size, max_blocks, num_blocks;
};

template <typename T>
__global__ void __launch_bounds__(NORM_THREADS)
qkv_finish_kernel(const QkvFinishParams p) {
  __shared__ float red[2][NORM_THREADS / 32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float* nul = nullptr;
  // blockIdx.y: part of the row.  Part 0 does q, k and v; the activation is spread over the others (over part 0
  // when there is only one), because it is most of the row and waits for nothing.
  const int act_parts = max(static_cast<int>(gridDim.y) - 1, 1), act_part = gridDim.y > 1 ? static_cast<int>(blockIdx.y) - 1 : 0;
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x) {
    T* y = static_cast<T*>(p.packed) + static_cast<long long>(row) * p.ld;
    if (act_part >= 0) {
      T* up_out = static_cast<T*>(p.act_out) + static_cast<long long>(row) * p.ld_act;
      const int stride = act_parts * NORM_THREADS * 8;
      for (int i = (act_part * NORM_THREADS + threadIdx.x) * 8; i < p.up_n; i += 2 * stride) {   // two loads in flight
        const int i2 = i + stride < p.up_n ? i + stride : i;
        float f[8], g[8];
        load8(y + p.up_off + i, f);
        load8(y + p.up_off + i2, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = act_row(f[j], p.act, y);
        store8(up_out + i, f);
        if (i2 != i) {
#pragma unroll
          for (int j = 0; j < 8; ++j) g[j] = act_row(g[j], p.act, y);
          store8(up_out + i2, g);
        }
      }
    }
    if (blockIdx.y > 0) continue;
    const int position = p.pos[row];
    float sq = 0.f, sk = 0.f;
    if (p.q_weight != nul)
      for (int i = threadIdx.x * 8; i < p.q_n; i += NORM_THREADS * 8) {
        float f[8];
        load8(y + p.q_off + i, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) sq += f[j] * f[j];
      }
    if (p.k_weight != nul)
      for (int i = threadIdx.x * 8; i < p.k_n; i += NORM_THREADS * 8) {
        float f[8];
        load8(y + p.k_off + i, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) sk += f[j] * f[j];
      }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    __syncthreads();                       // the previous row's sums have been read
    if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
    const int blk = p.block_table[static_cast<long long>(p.slots[row]) * p.max_blocks + position / p.block_size];
    const bool cached = blk >= 0 && blk < p.num_blocks;    // host validates; never write out of range
    const long long token = static_cast<long long>(blk) * p.block_size + position % p.block_size;
    if (cached)
      for (int i = threadIdx.x * 8; i < p.v_n; i += NORM_THREADS * 8) {
        float f[8];
        load8(y + p.v_off + i, f);
        store8(static_cast<T*>(p.v_cache) + token * p.v_n + i, f);
      }
    __syncthreads();
    sq = 0.f; sk = 0.f;
#pragma unroll
    for (int w = 0; w < NORM_THREADS / 32; ++w) { sq += red[0][w]; sk += red[1][w]; }
    float rq = 1.f;
    if (p.q_weight != nul) rq = 1.f / sqrtf(sq / static_cast<float>(p.q_count) + p.eps);
    if (p.temp_coef != 0.f)
      rq *= 1.f + p.temp_coef * logf(static_cast<float>(floor((position + 1) / p.temp_every)) + 1.f);
    if (p.q_weight != nul || p.temp_coef != 0.f)
      for (int i = threadIdx.x * 8; i < p.q_n; i += NORM_THREADS * 8) {
        float f[8], w[8];
        load8(y + p.q_off + i, f);
        if (p.q_weight != nul) load8(p.q_weight + i, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= p.q_weight != nul ? rq * w[j] : rq;
        store8(y + p.q_off + i, f);
      }
    if (cached) {
      const float rk = p.k_weight != nul ? 1.f / sqrtf(sk / static_cast<float>(p.k_count) + p.eps) : 1.f;
      for (int i = threadIdx.x * 8; i < p.k_n; i += NORM_THREADS * 8) {
        float f[8], w[8];
        load8(y + p.k_off + i, f);
        if (p.k_weight != nul) {
          load8(p.k_weight + i, w);
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] *= rk * w[j];
        }
        store8(static_cast<T*>(p.k_cache) + token * p.k_n + i, f);
      }
    }
  }
}

}  // namespace ft

using namespace ft;

FT_API int ft_rmsnorm_fwd(const void* x, const void* delta, const void* w, void* y, void* res_out,
                          float* rstd, int rows, int H, float eps, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(x && w && y, "ft_rmsnorm_fwd: null pointer");
  FT_REQUIRE(H % 8 == 0 && H <= NORM_THREADS * NORM_MAX_VEC * 8, "ft_rmsnorm_fwd: H=%d unsupported", H);
  if (rows <= 0) return FT_E_OK;
  const int grid = rows < sm_count(device) * 8 ? rows : sm_count(device) * 8;
  rmsnorm_fwd_kernel<<<grid, NORM_THREADS, 0, stream>>>(
      static_cast<const __nv_bfloat16*>(x), static_cast<const __nv_bfloat16*>(delta),
      static_cast<const __nv_bfloat16*>(w), static_cast<__nv_bfloat16*>(y),
      static_cast<__nv_bfloat16*>(res_out), rstd, rows, H, eps);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// Number of fp32 scratch rows ft_rmsnorm_bwd needs for `rows` (scratch = n * H floats).
FT_API int ft_rmsnorm_bwd_scratch_rows(int rows, int device) {
  const int cap = sm_count(device) * 2;
  return rows < cap ? (rows > 0 ? rows : 1) : cap;
}

// dw may be null (then scratch may be null too).  dw_flags: bit0 fp32 output, bit1 accumulate.
FT_API int ft_rmsnorm_bwd(const void* dy, const void* x, const void* w, const float* rstd,
                          const void* dres, void* dx, void* dw, float* scratch, int rows, int H,
                          int dw_flags, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(dy && x && w && rstd && dx, "ft_rmsnorm_bwd: null pointer");
  FT_REQUIRE(H % 8 == 0 && H <= NORM_THREADS * NORM_MAX_VEC * 8, "ft_rmsnorm_bwd: H=%d unsupported", H);
  FT_REQUIRE(!dw || scratch, "ft_rmsnorm_bwd: dw requested without scratch");
  if (rows <= 0) return FT_E_OK;
  const int grid = ft_rmsnorm_bwd_scratch_rows(rows, device);
  rmsnorm_bwd_kernel<<<grid, NORM_THREADS, 0, stream>>>(
      static_cast<const __nv_bfloat16*>(dy), static_cast<const __nv_bfloat16*>(x),
      static_cast<const __nv_bfloat16*>(w), rstd, static_cast<const __nv_bfloat16*>(dres),
      static_cast<__nv_bfloat16*>(dx), dw ? scratch : nullptr, rows, H);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  if (dw) {
    rmsnorm_dw_reduce_kernel<<<(H + DW_RED_COLS - 1) / DW_RED_COLS, DW_RED_COLS * DW_RED_WARPS, 0, stream>>>(scratch, dw, grid, H, dw_flags & 1,
                                                                  (dw_flags >> 1) & 1);
    FT_CUDA_CHECK(cudaGetLastError());
    count_launch();
  }
  return FT_E_OK;
}

FT_API int ft_rope(void* x, const float* cos_t, const float* sin_t, const int* pos, int T,
                   int n_rot_heads, int D, long long ld, int seq_len, int pos_offset, int interleaved,
                   int backward, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(x && cos_t && sin_t, "ft_rope: null pointer");
  FT_REQUIRE(D % 4 == 0 && ld % 4 == 0, "ft_rope: head_dim and row stride must be multiples of 4");
  FT_REQUIRE(pos || seq_len > 0, "ft_rope: need positions or seq_len");
  if (T <= 0 || n_rot_heads <= 0) return FT_E_OK;
  const long long work = static_cast<long long>(T) * n_rot_heads * (D / 4);
  if (D % 16 == 0 && ld % 8 == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0 &&
      (reinterpret_cast<uintptr_t>(cos_t) & 15) == 0 && (reinterpret_cast<uintptr_t>(sin_t) & 15) == 0)
    rope_vec_kernel<<<blocks_for(work / 4, 256, device), 256, 0, stream>>>(
        static_cast<__nv_bfloat16*>(x), cos_t, sin_t, pos, T, n_rot_heads, D, ld, seq_len, pos_offset,
        interleaved, backward ? -1.f : 1.f);
  else
    rope_kernel<<<blocks_for(work, 256, device), 256, 0, stream>>>(
        static_cast<__nv_bfloat16*>(x), cos_t, sin_t, pos, T, n_rot_heads, D, ld, seq_len, pos_offset,
        interleaved, backward ? -1.f : 1.f);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

FT_API int ft_swiglu_fwd(const void* gu, void* out, long long T, int F, long long ld_gu, int act,
                         int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(gu && out, "ft_swiglu_fwd: null pointer");
  FT_REQUIRE(F % 8 == 0 && ld_gu % 8 == 0, "ft_swiglu_fwd: F must be a multiple of 8");
  if (T <= 0) return FT_E_OK;
  swiglu_fwd2_kernel<<<blocks_for(T * (F / 8) / 2 + 1, 256, device), 256, 0, stream>>>(
      static_cast<const __nv_bfloat16*>(gu), static_cast<__nv_bfloat16*>(out), T, F, ld_gu, act);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

FT_API int ft_swiglu_bwd(const void* dy, const void* gu, void* dgu, long long T, int F, long long ld_gu,
                         int act, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(dy && gu && dgu, "ft_swiglu_bwd: null pointer");
  FT_REQUIRE(F % 8 == 0 && ld_gu % 8 == 0, "ft_swiglu_bwd: F must be a multiple of 8");
  if (T <= 0) return FT_E_OK;
  swiglu_bwd2_kernel<<<blocks_for(T * (F / 8) / 2 + 1, 256, device), 256, 0, stream>>>(
      static_cast<const __nv_bfloat16*>(dy), static_cast<const __nv_bfloat16*>(gu),
      static_cast<__nv_bfloat16*>(dgu), T, F, ld_gu, act);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

FT_API int ft_embedding_fwd(const long long* ids, const void* w, void* out, int T, int H, int vocab,
                            int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(ids && w && out && H % 8 == 0, "ft_embedding_fwd: bad arguments");
  if (T <= 0) return FT_E_OK;
  const int grid = T < sm_count(device) * 16 ? T : sm_count(device) * 16;
  embedding_fwd_kernel<<<grid, 128, 0, stream>>>(ids, static_cast<const __nv_bfloat16*>(w),
                                                 static_cast<__nv_bfloat16*>(out), T, H, vocab);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

FT_API int ft_embedding_bwd(const long long* ids, const void* dy, void* dw, int T, int H, int vocab,
                            int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(ids && dy && dw && H % 2 == 0, "ft_embedding_bwd: bad arguments");
  if (T <= 0) return FT_E_OK;
  const int grid = T < sm_count(device) * 16 ? T : sm_count(device) * 16;
  embedding_bwd_kernel<<<grid, 128, 0, stream>>>(ids, static_cast<const __nv_bfloat16*>(dy),
                                                 static_cast<__nv_bfloat16*>(dw), T, H, vocab);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// Dynamic tanh: y[rows, H] = (tanh(alpha x) w + b) * scale.  x: fp32 [rows, ldx], or with ids (int64
// [rows]) the rows table[ids] of a bf16 (in_bf16) or fp32 table [vocab, ldx], which are then also
// written to x_out (fp32 [rows, H]).  y: bf16, or fp32 with out_f32.  alpha: one fp32 on the device.
FT_API int ft_dyt_fwd(const void* x, const long long* ids, int vocab, int in_bf16, float* x_out, const float* alpha,
                      const float* w, const float* b, void* y, int out_f32, int rows, int H, long long ldx, long long ldy,
                      float scale, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(x && alpha && w && b && y, "ft_dyt_fwd: null pointer");
  FT_REQUIRE(H > 0 && H % 8 == 0 && ldx % 8 == 0 && ldy % 8 == 0 && ldx >= H && ldy >= H, "ft_dyt_fwd: H=%d and strides must be multiples of 8", H);
  FT_REQUIRE(((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(w) |
               reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(x_out)) & 15) == 0, "ft_dyt_fwd: pointers must be 16-byte aligned");
  FT_REQUIRE(!ids || vocab > 0, "ft_dyt_fwd: a gather needs the table size");
  if (rows <= 0) return FT_E_OK;
  const int gx = (H / 8 + NORM_THREADS - 1) / NORM_THREADS;
  int gy = sm_count(device) * 8 / gx;
  if (gy < 1) gy = 1;
  if (gy > rows) gy = rows;
  const dim3 grid(gx, gy);
#define FT_DYT(TI, TO)                                                                                             \
  dyt_kernel<TI, TO><<<grid, NORM_THREADS, 0, stream>>>(static_cast<const TI*>(x), ids, vocab, x_out, alpha, w, b, \
                                                        static_cast<TO*>(y), rows, H, ldx, ldy, scale)
  if (in_bf16) {
    if (out_f32) FT_DYT(__nv_bfloat16, float); else FT_DYT(__nv_bfloat16, __nv_bfloat16);
  } else {
    if (out_f32) FT_DYT(float, float); else FT_DYT(float, __nv_bfloat16);
  }
#undef FT_DYT
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// The pass between a packed input projection and its attention (see qkv_finish_kernel).  packed, caches
// and act_out are bf16, or fp32 with f32.  Offsets and sizes in elements, multiples of 8.  row_parts: blocks that
// share a row (0: chosen here).
FT_API int ft_qkv_finish(void* packed, long long ld, const int* pos, const int* slots, const int* block_table, void* k_cache,
                         void* v_cache, const float* q_weight, const float* k_weight, void* act_out, long long ld_act,
                         int rows, int q_off, int q_n, int k_off, int k_n, int v_off, int v_n, int up_off, int up_n,
                         int q_count, int k_count, float eps, float temp_coef, float temp_every, int act, int f32,
                         int block_size, int max_blocks, int num_blocks, int row_parts, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(packed && pos && slots && block_table && k_cache && v_cache, "ft_qkv_finish: null pointer");
  FT_REQUIRE(((q_off | q_n | k_off | k_n | v_off | v_n | up_off | up_n) & 7) == 0 && ld % 8 == 0 && ld_act % 8 == 0,
             "ft_qkv_finish: offsets, sizes and strides must be multiples of 8");
  FT_REQUIRE(q_n > 0 && k_n > 0 && v_n > 0 && up_n >= 0 && q_off >= 0 && k_off >= 0 && v_off >= 0 && up_off >= 0 &&
                 q_off + q_n <= ld && k_off + k_n <= ld && v_off + v_n <= ld && up_off + up_n <= ld && (up_n == 0 || (act_out && up_n <= ld_act)),
             "ft_qkv_finish: a segment lies outside the row");
  FT_REQUIRE(((reinterpret_cast<uintptr_t>(packed) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) |
               reinterpret_cast<uintptr_t>(q_weight) | reinterpret_cast<uintptr_t>(k_weight) | reinterpret_cast<uintptr_t>(act_out)) & 15) == 0,
             "ft_qkv_finish: pointers must be 16-byte aligned");
  FT_REQUIRE(block_size > 0 && max_blocks > 0 && num_blocks > 0 && q_count > 0 && k_count > 0 && temp_every > 0.f && act >= 0 && act <= 2,
             "ft_qkv_finish: bad argument");
  if (rows <= 0) return FT_E_OK;
  QkvFinishParams p;
  p.packed = packed; p.ld = ld; p.pos = pos; p.slots = slots; p.block_table = block_table;
  p.k_cache = k_cache; p.v_cache = v_cache; p.q_weight = q_weight; p.k_weight = k_weight;
  p.act_out = act_out; p.ld_act = ld_act; p.rows = rows;
  p.q_off = q_off; p.q_n = q_n; p.k_off = k_off; p.k_n = k_n; p.v_off = v_off; p.v_n = v_n;
  p.up_off = up_off; p.up_n = up_n; p.q_count = q_count; p.k_count = k_count;
  p.eps = eps; p.temp_coef = temp_coef; p.temp_every = temp_every;
  p.act = act; p.block_size = block_size; p.max_blocks = max_blocks; p.num_blocks = num_blocks;
  // a batch that does not fill the GPU is cut into one more part per pass of a block over the activation
  const int wave = sm_count(device) * 8;
  if (row_parts <= 0) {
    row_parts = up_n > 0 ? 1 + (up_n + NORM_THREADS * 8 - 1) / (NORM_THREADS * 8) : 1;
    if (row_parts > wave / rows) row_parts = wave / rows > 1 ? wave / rows : 1;
  }
  if (row_parts > 64) row_parts = 64;
  int per_part = wave / row_parts > 0 ? wave / row_parts : 1;
  const dim3 grid(rows < per_part ? rows : per_part, row_parts);
  if (f32) qkv_finish_kernel<float><<<grid, NORM_THREADS, 0, stream>>>(p);
  else qkv_finish_kernel<__nv_bfloat16><<<grid, NORM_THREADS, 0, stream>>>(p);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// ---------------------------------------------------------------------------------------------
// RMSNorm backward for callers that must not allocate (declaration and contract: ft_noalloc.h).
// The partial sums of dw go to this fixed array instead of caller-provided scratch.  In host
// code the name below is only a handle for cudaGetSymbolAddress, never a device pointer.
#include "ft_noalloc.h"

static __device__ __align__(256) float g_rmsnorm_noalloc_scratch[FT_NOALLOC_RMSNORM_ROWS * FT_NOALLOC_RMSNORM_MAX_H];

FT_API int ft_rmsnorm_bwd_noalloc(const void* dy, const void* x, const void* w, const float* rstd,
                                  const void* dres, void* dx, void* dw, int rows, int H, int dw_flags,
                                  int device, cudaStream_t stream) {
  FT_REQUIRE(dy && x && w && rstd && dx, "ft_rmsnorm_bwd_noalloc: null pointer");
  FT_REQUIRE(device >= 0 && device < 64, "ft_rmsnorm_bwd_noalloc: bad device %d", device);
  FT_REQUIRE(H > 0 && H % 8 == 0, "ft_rmsnorm_bwd_noalloc: H=%d must be a positive multiple of 8", H);
  if (H > FT_NOALLOC_RMSNORM_MAX_H) {
    set_last_error("ft_rmsnorm_bwd_noalloc: H=%d exceeds the fixed scratch (max %d); use ft_rmsnorm_bwd "
                   "with caller-provided scratch", H, FT_NOALLOC_RMSNORM_MAX_H);
    return FT_E_TOO_LARGE;
  }
  // The kernels below launch on the calling thread's current device, and the scratch address
  // belongs to `device`: the two must be the same GPU.  (Checked, not switched: switching would
  // have to be undone on every error path, and a caller that cannot allocate usually also wants
  // no hidden device changes.)
  int cur = -1;
  FT_CUDA_CHECK(cudaGetDevice(&cur));
  FT_REQUIRE(cur == device, "ft_rmsnorm_bwd_noalloc: device %d must be the current device (current is %d)",
             device, cur);
  if (rows <= 0) return FT_E_OK;
  // Once per device, with that device current: resolve the device address of the array.  Two
  // threads that race here both store the same value, so the unsynchronised write is benign.
  static float* scratch_of[64] = {nullptr};
  if (!scratch_of[device]) {
    float* ptr = nullptr;
    const cudaError_t e = cudaGetSymbolAddress(reinterpret_cast<void**>(&ptr), g_rmsnorm_noalloc_scratch);
    if (e != cudaSuccess || !ptr) {
      set_last_error("ft_rmsnorm_bwd_noalloc: cudaGetSymbolAddress failed: %s", cudaGetErrorString(e));
      return FT_E_CUDA;
    }
    scratch_of[device] = ptr;
  }
  float* scratch = scratch_of[device];
  const int grid = rows < FT_NOALLOC_RMSNORM_ROWS ? rows : FT_NOALLOC_RMSNORM_ROWS;
  // every partial row [0, grid) x [0, H) is written by the first kernel before the second reads
  // it, so the previous call's contents never leak into the result
  rmsnorm_bwd_kernel<<<grid, NORM_THREADS, 0, stream>>>(
      static_cast<const __nv_bfloat16*>(dy), static_cast<const __nv_bfloat16*>(x),
      static_cast<const __nv_bfloat16*>(w), rstd, static_cast<const __nv_bfloat16*>(dres),
      static_cast<__nv_bfloat16*>(dx), dw ? scratch : nullptr, rows, H);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  if (dw) {
    rmsnorm_dw_reduce_kernel<<<(H + DW_RED_COLS - 1) / DW_RED_COLS, DW_RED_COLS * DW_RED_WARPS, 0, stream>>>(scratch, dw, grid, H, dw_flags & 1,
                                                                  (dw_flags >> 1) & 1);
    FT_CUDA_CHECK(cudaGetLastError());
    count_launch();
  }
  return FT_E_OK;
}
