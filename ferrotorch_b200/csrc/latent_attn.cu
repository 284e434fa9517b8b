// Latent attention over the paged cache: a token's cached row is its latent c (of `rank` elements) followed by one rotated
// key part that all heads share; keys and values of a head are linear in c.
//
//   ft_latent_finish   everything between the packed projection [ q heads | latent | rotated key part | .. ] and the
//                      attention: RMS norm of the latent, rotation of the key part and of every head's rotated
//                      query part (neighbouring elements are pairs), the row into its cache page
#include <initializer_list>

#include "row_vec.cuh"

namespace ft {

constexpr int LF_THREADS = 128;

struct LatentFinishParams {
  void* packed;             // [rows, ld]
  void* q_lat;              // [n_lat, H, ldq_head]: rows 0 .. n_lat - 1 put their rotated query parts here, behind the latent part
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

// One block per row: the first warp takes the latent and the key part, the others the queries.
template <typename T>
__global__ void __launch_bounds__(LF_THREADS)
latent_finish_kernel(const LatentFinishParams p) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int width = p.rank_pad + p.rot_pad;
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x) {
    T* y = static_cast<T*>(p.packed) + static_cast<long long>(row) * p.ld;
    const int position = p.pos[row];
    const float2* cs = p.table + static_cast<long long>(min(position, p.positions - 1)) * p.half;
    if (warp == 0) {
      const int page = position / p.block_size;
      const int blk = page < p.max_blocks ? p.block_table[static_cast<long long>(p.slots[row]) * p.max_blocks + page] : -1;
      T* dst = blk >= 0 && blk < p.num_blocks
                   ? static_cast<T*>(p.cache) + (static_cast<long long>(blk) * p.block_size + position % p.block_size) * width : nullptr;
      T* c = y + p.c_off;
      float sum = 0.f;
      for (int i = lane * 8; i < p.rank_pad; i += 256) {
        float f[8];
        load8(c + i, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum += f[e] * f[e];
      }
      const float r = 1.f / sqrtf(warp_sum(sum) / static_cast<float>(p.rank) + p.eps);
      for (int i = lane * 8; i < width; i += 256) {
        float f[8];
        load8(c + i, f);
        if (i < p.rank_pad) {
          float w[8];
          load8(p.weight + i, w);
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] *= r * w[e];
        } else {
          rotate8(f, i - p.rank_pad, cs, p.half);
        }
        store8(c + i, f);
        if (dst) store8(dst + i, f);
      }
    } else {
      const int units = p.rot_pad / 8;
      for (int u = threadIdx.x - 32; u < p.H * units; u += LF_THREADS - 32) {
        const int h = u / units, d = (u - h * units) * 8;
        T* q = y + p.q_off + static_cast<long long>(h) * p.q_head + p.q_rot + d;
        float f[8];
        load8(q, f);
        rotate8(f, d, cs, p.half);
        store8(row < p.n_lat ? static_cast<T*>(p.q_lat) + (static_cast<long long>(row) * p.H + h) * width + p.rank_pad + d : q, f);
      }
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
// 8.  Rows n_lat .. keep their rotated query parts in place, the rows ahead of them put theirs into q_lat.
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
  const int cap = sm_count(device) * 16, grid = rows < cap ? rows : cap;
  if (f32) latent_finish_kernel<float><<<grid, LF_THREADS, 0, stream>>>(p);
  else latent_finish_kernel<__nv_bfloat16><<<grid, LF_THREADS, 0, stream>>>(p);
  FT_CUDA_CHECK(cudaGetLastError());
  count_launch();
  return FT_E_OK;
}
