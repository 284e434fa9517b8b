// Row kernels of decoders whose residual is several fp32 streams (hyper-connections), and of n-gram embeddings:
//
//   ft_stream_step    all streams at once after a sublayer, x_t <- sum_s mix[s, t] x_s + out[t] y, the weighted sum
//                     u = sum_t in[t] x_t that the next sublayer reads, and its RMS norm, in one pass over the row.  y is a
//                     dense row, the weighted outputs of a token's experts (still sorted by expert), or both.
//   ft_embed_bigram   scaled token embedding plus a row of a table hashed from the previous and the present token; the
//                     previous token of a portion comes from the page that holds the position before it, and every
//                     row leaves its own token there.  Also writes the first sublayer's normed input.
//   ft_softcap        cap * tanh(z / cap) over rows of logits
//
// Arithmetic is fp32.
#include <initializer_list>

#include "row_vec.cuh"

namespace ft {

constexpr int ST_KEEP = 4;        // vectors of four elements a thread keeps
constexpr int ST_MAX_THREADS = 1024;

__device__ __forceinline__ void load4(const float* p, float (&f)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&f)[4]) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
__device__ __forceinline__ void store4(float* p, const float (&f)[4]) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&f)[4]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
}

// Sum over the block; `red` has one float per warp.  Every thread receives the sum.
__device__ __forceinline__ float block_total(float v, float* red) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  v = warp_sum(v);
  __syncthreads();                       // the previous total has been read
  if (lane == 0) red[warp] = v;
  __syncthreads();
  v = 0.f;
  for (int w = 0; w < warps; ++w) v += red[w];
  return v;
}

// The normed row from the kept vectors.
template <typename TO>
__device__ __forceinline__ void store_normed(const float (&u)[ST_KEEP][4], float sum, const float* w, TO* h, int H, int count, float eps) {
  const float r = 1.f / sqrtf(sum / static_cast<float>(count) + eps);
#pragma unroll
  for (int k = 0; k < ST_KEEP; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 4;
    if (i >= H) continue;
    float f[4];
    load4(w + i, f);
#pragma unroll
    for (int e = 0; e < 4; ++e) f[e] = u[k][e] * r * f[e];
    store4(h + i, f);
  }
}

struct StreamParams {
  const float* x;           // stream s of row r: x + r * ldx + s * lds (lds 0: all streams are the same row)
  const long long* ids;     // row i reads row ids[i] of everything (null: i)
  float* x_out;             // [rows, S, H]; may be x; null: not written
  const float* mix;         // [S, S], [from, to]
  const float* out;         // [S]
  const float* in;          // [S]
  const void* y;            // [n_src, ldy] or null
  const void* terms;        // [term_rows, ldt]: y gains weight[r, j] * terms[where[r, j]]; where < 0: weight[r, j] * self[r]
  const int* where;
  const float* weight;      // null: ones
  const void* self;         // [n_src, ldself]
  const float* w;           // norm weight
  void* h;                  // [rows, ldh]
  long long ldx, lds, ldy, ldt, ldself, ldh;
  int rows, n_src, S, H, count, n_terms, term_rows;
  float eps;
};

template <typename T, int SM>
__global__ void __launch_bounds__(ST_MAX_THREADS)
stream_step_kernel(const StreamParams p) {
  __shared__ float red[32], s_mix[SM * SM], s_out[SM], s_in[SM];
  for (int i = threadIdx.x; i < p.S * p.S; i += blockDim.x) s_mix[(i / p.S) * SM + i % p.S] = p.mix[i];
  if (static_cast<int>(threadIdx.x) < p.S) {
    s_out[threadIdx.x] = p.out[threadIdx.x];
    s_in[threadIdx.x] = p.in[threadIdx.x];
  }
  __syncthreads();
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x) {
    long long src = row;
    if (p.ids) {
      src = p.ids[row];
      if (src < 0 || src >= p.n_src) src = 0;    // host validates; never read out of range
    }
    const float* xr = p.x + src * p.ldx;
    float* xo = p.x_out ? p.x_out + static_cast<long long>(row) * p.S * p.H : nullptr;
    float u[ST_KEEP][4];
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < ST_KEEP; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 4;
      if (i >= p.H) continue;
      float x[SM][4], y[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < p.S) load4(xr + s * p.lds + i, x[s]);
      if (p.y) load4(static_cast<const T*>(p.y) + src * p.ldy + i, y);
      for (int j = 0; j < p.n_terms; ++j) {
        const int t = p.where[src * p.n_terms + j];
        const float g = p.weight ? p.weight[src * p.n_terms + j] : 1.f;
        if (t >= p.term_rows || (t < 0 && !p.self)) continue;
        float f[4];
        load4(t < 0 ? static_cast<const T*>(p.self) + src * p.ldself + i : static_cast<const T*>(p.terms) + static_cast<long long>(t) * p.ldt + i, f);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] += g * f[e];
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) u[k][e] = 0.f;
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= p.S) continue;
        float v[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = s_out[t] * y[e];
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < p.S) {
            const float c = s_mix[s * SM + t];
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] += c * x[s][e];
          }
        if (xo) store4(xo + static_cast<long long>(t) * p.H + i, v);
#pragma unroll
        for (int e = 0; e < 4; ++e) u[k][e] += s_in[t] * v[e];
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) sum += u[k][e] * u[k][e];
    }
    sum = block_total(sum, red);
    store_normed(u, sum, p.w, static_cast<T*>(p.h) + static_cast<long long>(row) * p.ldh, p.H, p.count, p.eps);
  }
}

struct EmbedParams {
  const long long* tokens;
  const int* pos;
  const int* starts;        // position of the first row of the row's portion
  const int* slots;
  const int* block_table;
  int* token_pages;         // [num_blocks, block_size]
  const void* table;        // [vocab, ld]
  const void* bigram;       // [buckets + 1, ld]
  const float* in;          // [S]: u = sum(in) x
  const float* w;
  float* x;                 // [rows, H]
  void* h;                  // [rows, H]
  long long ld, mul_prev, mul_cur;
  int rows, S, H, count, vocab, buckets, block_size, max_blocks, num_blocks;
  float scale, eps;
};

constexpr int EB_KEEP = 2;        // vectors of eight elements a thread keeps

template <typename T>
__global__ void __launch_bounds__(ST_MAX_THREADS)
embed_bigram_kernel(const EmbedParams p) {
  __shared__ float red[32];
  float in = 0.f;
  for (int s = 0; s < p.S; ++s) in += p.in[s];
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x) {
    long long token = p.tokens[row];
    if (token < 0 || token >= p.vocab) token = 0;
    const T* er = static_cast<const T*>(p.table) + token * p.ld;
    float u[EB_KEEP][8];
#pragma unroll
    for (int k = 0; k < EB_KEEP; ++k) {              // the token's row is on its way while the previous token is looked up
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      if (i < p.H) load8(er + i, u[k]);
    }
    const int pos = p.pos[row];
    const int* bt = p.block_table + static_cast<long long>(p.slots[row]) * p.max_blocks;
    auto page_of = [&](int q) -> long long {
      const int page = q / p.block_size;
      const int blk = page < p.max_blocks ? bt[page] : -1;
      return blk < 0 || blk >= p.num_blocks ? -1 : static_cast<long long>(blk) * p.block_size + q % p.block_size;
    };
    long long bucket = p.buckets;
    if (pos > 0) {
      long long prev = 0;
      if (pos > p.starts[row]) prev = p.tokens[row - 1];
      else {
        const long long at = page_of(pos - 1);
        if (at >= 0) prev = p.token_pages[at];
      }
      bucket = (prev * p.mul_prev + token * p.mul_cur) % p.buckets;
      if (bucket < 0) bucket += p.buckets;
    }
    const T* br = static_cast<const T*>(p.bigram) + bucket * p.ld;
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < EB_KEEP; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      if (i >= p.H) continue;
      float b[8];
      load8(br + i, b);
#pragma unroll
      for (int e = 0; e < 8; ++e) b[e] = u[k][e] * p.scale + b[e];
      store8(p.x + static_cast<long long>(row) * p.H + i, b);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        u[k][e] = in * b[e];
        sum += u[k][e] * u[k][e];
      }
    }
    if (threadIdx.x == 0) {                          // no row reads a page place that a row of the same step writes
      const long long at = page_of(pos);
      if (at >= 0) p.token_pages[at] = static_cast<int>(token);
    }
    sum = block_total(sum, red);
    const float r = 1.f / sqrtf(sum / static_cast<float>(p.count) + p.eps);
    T* h = static_cast<T*>(p.h) + static_cast<long long>(row) * p.H;
#pragma unroll
    for (int k = 0; k < EB_KEEP; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      if (i >= p.H) continue;
      float w[8];
      load8(p.w + i, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) w[e] = u[k][e] * r * w[e];
      store8(h + i, w);
    }
  }
}

__global__ void softcap_kernel(float* __restrict__ z, long long n, float cap, float inv) {
  for (long long i = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) * 4; i < n; i += static_cast<long long>(gridDim.x) * blockDim.x * 4) {
    float f[4];
    load4(z + i, f);
#pragma unroll
    for (int e = 0; e < 4; ++e) f[e] = cap * tanhf(f[e] * inv);
    store4(z + i, f);
  }
}

static bool st_aligned(std::initializer_list<const void*> ps) {
  uintptr_t v = 0;
  for (const void* p : ps) v |= reinterpret_cast<uintptr_t>(p);
  return (v & 15) == 0;
}

// Threads of a block for rows of H elements: two vectors a thread where that leaves a few warps, never more than ST_KEEP.
static int stream_threads(int H) {
  int t = (H / 4 + 1) / 2;
  t = (t + 31) / 32 * 32;
  return t < 64 ? 64 : (t > ST_MAX_THREADS ? ST_MAX_THREADS : t);
}

}  // namespace ft

using namespace ft;

// One step of S fp32 streams (see StreamParams): x [n_src, ldx] (stream stride lds, 0: one row for all), x_out [rows, S, H] or
// null (may be x without ids), y / terms / self / h bf16, or fp32 with f32.  H: padded width, a multiple of 8 up to 16384,
// count: true width.  where int32 and weight fp32 [n_src, n_terms].
FT_API int ft_stream_step(const float* x, long long ldx, long long lds, const long long* ids, int n_src, float* x_out, const float* mix,
                          const float* out, const float* in, int S, const void* y, long long ldy, const void* terms, long long ldt,
                          int term_rows, const int* where, const float* weight, int n_terms, const void* self, long long ldself,
                          const float* w, void* h, long long ldh, int rows, int H, int count, float eps, int f32, int device,
                          cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(x && mix && out && in && w && h, "ft_stream_step: null pointer");
  FT_REQUIRE(S >= 1 && S <= 16, "ft_stream_step: %d streams (1 to 16)", S);
  FT_REQUIRE(H > 0 && H % 8 == 0 && H <= ST_KEEP * 4 * ST_MAX_THREADS && count > 0 && count <= H, "ft_stream_step: rows of %d", H);
  FT_REQUIRE(((ldx | lds | ldy | ldt | ldself | ldh) & 7) == 0 && ldh >= H && (lds == 0 || lds >= H), "ft_stream_step: strides must be multiples of 8");
  FT_REQUIRE(n_terms == 0 || (n_terms > 0 && terms && where && ldt >= H && term_rows > 0), "ft_stream_step: terms without their rows");
  FT_REQUIRE(st_aligned({x, x_out, y, terms, self, w, h}), "ft_stream_step: pointers must be 16-byte aligned");
  FT_REQUIRE(n_src > 0 && (ids || rows <= n_src), "ft_stream_step: %d source rows", n_src);
  if (rows <= 0) return FT_E_OK;
  StreamParams p;
  p.x = x; p.ids = ids; p.x_out = x_out; p.mix = mix; p.out = out; p.in = in; p.y = y; p.terms = terms; p.where = where;
  p.weight = weight; p.self = self; p.w = w; p.h = h;
  p.ldx = ldx; p.lds = lds; p.ldy = ldy; p.ldt = ldt; p.ldself = ldself; p.ldh = ldh;
  p.rows = rows; p.n_src = n_src; p.S = S; p.H = H; p.count = count; p.n_terms = n_terms; p.term_rows = term_rows; p.eps = eps;
  const int cap = sm_count(device) * 32, grid = rows < cap ? rows : cap, threads = stream_threads(H);
#define FT_ST(T)                                                               \
  if (S <= 2) stream_step_kernel<T, 2><<<grid, threads, 0, stream>>>(p);       \
  else if (S <= 4) stream_step_kernel<T, 4><<<grid, threads, 0, stream>>>(p);  \
  else if (S <= 8) stream_step_kernel<T, 8><<<grid, threads, 0, stream>>>(p);  \
  else stream_step_kernel<T, 16><<<grid, threads, 0, stream>>>(p)
  if (f32) { FT_ST(float); } else { FT_ST(__nv_bfloat16); }
#undef FT_ST
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// Embedding of a ragged batch with a hashed table of token pairs (see embed_bigram_kernel): x fp32 [rows, H], h [rows, H] the RMS
// norm of sum(in) x.  table [vocab, ld] and bigram [buckets + 1, ld] are bf16, or fp32 with f32.
FT_API int ft_embed_bigram(const long long* tokens, const int* pos, const int* starts, const int* slots, const int* block_table,
                           int* token_pages, const void* table, const void* bigram, long long ld, int vocab, int buckets,
                           long long mul_prev, long long mul_cur, float scale, const float* in, int S, const float* w, float* x,
                           void* h, int rows, int H, int count, float eps, int f32, int block_size, int max_blocks, int num_blocks,
                           int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(tokens && pos && starts && slots && block_table && token_pages && table && bigram && in && w && x && h, "ft_embed_bigram: null pointer");
  FT_REQUIRE(H > 0 && H % 8 == 0 && H <= EB_KEEP * 8 * ST_MAX_THREADS && count > 0 && count <= H && ld >= H && ld % 8 == 0, "ft_embed_bigram: rows of %d", H);
  FT_REQUIRE(vocab > 0 && buckets > 0 && S > 0 && block_size > 0 && max_blocks > 0 && num_blocks > 0, "ft_embed_bigram: bad shape");
  FT_REQUIRE(st_aligned({table, bigram, w, x, h}), "ft_embed_bigram: pointers must be 16-byte aligned");
  if (rows <= 0) return FT_E_OK;
  EmbedParams p;
  p.tokens = tokens; p.pos = pos; p.starts = starts; p.slots = slots; p.block_table = block_table; p.token_pages = token_pages;
  p.table = table; p.bigram = bigram; p.in = in; p.w = w; p.x = x; p.h = h; p.ld = ld; p.mul_prev = mul_prev; p.mul_cur = mul_cur;
  p.rows = rows; p.S = S; p.H = H; p.count = count; p.vocab = vocab; p.buckets = buckets; p.block_size = block_size;
  p.max_blocks = max_blocks; p.num_blocks = num_blocks; p.scale = scale; p.eps = eps;
  const int cap = sm_count(device) * 32, grid = rows < cap ? rows : cap;
  int threads = (H / 8 + EB_KEEP - 1) / EB_KEEP;
  threads = threads < 64 ? 64 : (threads + 31) / 32 * 32;
  if (f32) embed_bigram_kernel<float><<<grid, threads, 0, stream>>>(p);
  else embed_bigram_kernel<__nv_bfloat16><<<grid, threads, 0, stream>>>(p);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}

// z[0 .. n - 1] = cap * tanh(z / cap) in place, fp32, n a multiple of 4.
FT_API int ft_softcap(float* z, long long n, float cap, int device, cudaStream_t stream) {
  if (int _rc = ft::ensure_device(device)) return _rc;
  FT_REQUIRE(z && n % 4 == 0 && st_aligned({z}) && cap > 0.f, "ft_softcap: %lld elements, cap %g", n, cap);
  if (n <= 0) return FT_E_OK;
  softcap_kernel<<<blocks_for(n / 4, 256, device), 256, 0, stream>>>(z, n, cap, 1.f / cap);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}
