// Latent attention with per-layer sizes: what surrounds the products and the attention kernels (mla.cu for
// decode rows, attn_bias.cu for prompts).
//
//   latent_prepare_kernel   norms of the query and key latents, rotation of the shared key part, cache write
//   latent_queries_kernel   rotation of every head's rotated query part, in place or into absorbed rows
//   latent_gather_kernel    the pages that prompt portions see, one after the other
#include "api.h"
#include "sm100.cuh"

namespace b200 {

typedef __nv_bfloat16 bf16;

template <typename T> struct Lat4;
template <> struct Lat4<float> {
  static __device__ __forceinline__ float4 get(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void put(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Lat4<bf16> {
  static __device__ __forceinline__ float4 get(const bf16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
  }
  static __device__ __forceinline__ void put(bf16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  }
};
__device__ __forceinline__ float lat_to_f(float v) { return v; }
__device__ __forceinline__ float lat_to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void lat_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void lat_put(bf16* p, float v) { *p = __float2bfloat16(v); }

// One warp per token. Values beyond a latent's size (up to the next multiple of 8) are zeros in down and in
// the weights. kKeep: groups of 128 values kept in registers between the two passes over the query latent.
template <typename T>
__global__ void __launch_bounds__(128) latent_prepare_kernel(B200LatentPrep p) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= p.T) return;
  const T* row = reinterpret_cast<const T*>(p.down) + (size_t)t * p.ldd;
  const int64_t slot = reinterpret_cast<const int64_t*>(p.slots)[t];
  T* page = reinterpret_cast<T*>(p.cache) + (slot < 0 ? 0 : slot) * (int64_t)p.row;
  auto normed = [&](const T* src, const float* w, T* dst, int n) {
    static constexpr int kKeep = 4;
    const int n8 = (n + 7) & ~7;
    float4 keep[kKeep];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < kKeep; ++c) {
      const int i = c * 128 + lane * 4;
      keep[c] = i < n8 ? Lat4<T>::get(src + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += keep[c].x * keep[c].x + keep[c].y * keep[c].y + keep[c].z * keep[c].z + keep[c].w * keep[c].w;
    }
    for (int i = kKeep * 128 + lane * 4; i < n8; i += 128) {
      const float4 v = Lat4<T>::get(src + i);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = 1.f / sqrtf(ss / (float)n + p.eps);
    auto put = [&](int i, float4 v) {
      const float4 g = *reinterpret_cast<const float4*>(w + i);
      Lat4<T>::put(dst + i, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
    };
#pragma unroll
    for (int c = 0; c < kKeep; ++c)
      if (c * 128 + lane * 4 < n8) put(c * 128 + lane * 4, keep[c]);
    for (int i = kKeep * 128 + lane * 4; i < n8; i += 128) put(i, Lat4<T>::get(src + i));
  };
  normed(row, p.q_norm, reinterpret_cast<T*>(p.cq) + (size_t)t * p.ldcq, p.q_rank);
  if (slot < 0) return;
  normed(row + p.kv_col, p.kv_norm, page, p.rank);
  const int half = p.rot / 2;
  const float* cs = p.cos_sin + (size_t)reinterpret_cast<const int64_t*>(p.positions)[t] * p.rot;
  for (int i = lane; i < half; i += 32) {
    const float u = lat_to_f(row[p.rot_col + i]), v = lat_to_f(row[p.rot_col + half + i]), c = cs[i], s = cs[half + i];
    lat_put(page + p.rankp + i, u * c - v * s);
    lat_put(page + p.rankp + half + i, v * c + u * s);
  }
}

// A thread turns VEC pairs of one head. Rows t < absorbed go to the rotated columns of qabs.
template <typename T, int VEC>
__global__ void __launch_bounds__(128) latent_queries_kernel(T* q, long long ldq, const int64_t* positions, const float* cos_sin,
                                                             int H, int qn, int qw, int rot, T* qabs, int rankp, int row,
                                                             int absorbed, int T_) {
  pdl_wait();
  pdl_launch_dependents();
  const int half = rot / 2, per = half / VEC, n = H * per, t = blockIdx.y * gridDim.z + blockIdx.z;
  if (t >= T_) return;
  const float* cs = cos_sin + (size_t)positions[t] * rot;
  for (int x = blockIdx.x * 128 + threadIdx.x; x < n; x += gridDim.x * 128) {
    const int h = x / per, i = (x - h * per) * VEC;
    T* src = q + (size_t)t * ldq + (size_t)h * qw + qn;
    T* dst = t < absorbed ? qabs + ((size_t)t * H + h) * row + rankp : src;
    if constexpr (VEC == 4) {
      const float4 u = Lat4<T>::get(src + i), v = Lat4<T>::get(src + half + i);
      const float4 c = *reinterpret_cast<const float4*>(cs + i), s = *reinterpret_cast<const float4*>(cs + half + i);
      Lat4<T>::put(dst + i, make_float4(u.x * c.x - v.x * s.x, u.y * c.y - v.y * s.y, u.z * c.z - v.z * s.z, u.w * c.w - v.w * s.w));
      Lat4<T>::put(dst + half + i,
                   make_float4(v.x * c.x + u.x * s.x, v.y * c.y + u.y * s.y, v.z * c.z + u.z * s.z, v.w * c.w + u.w * s.w));
    } else {
      const float u = lat_to_f(src[i]), v = lat_to_f(src[half + i]), c = cs[i], s = cs[half + i];
      lat_put(dst + i, u * c - v * s);
      lat_put(dst + half + i, v * c + u * s);
    }
  }
}

// dense page base[r] + i = page first[r] + i of request r. page_bytes: a multiple of 16.
__global__ void __launch_bounds__(128) latent_gather_kernel(const uint8_t* cache, const int32_t* block_table, int max_blocks,
                                                            const int32_t* seq_lens, const int32_t* first, const int32_t* base,
                                                            int block_size, long long page_bytes, uint8_t* dense) {
  pdl_wait();
  pdl_launch_dependents();
  const int r = blockIdx.y, bi = blockIdx.x;
  if (bi < first[r] || bi >= (seq_lens[r] + block_size - 1) / block_size) return;
  const int blk = max(block_table[(size_t)r * max_blocks + bi], 0);
  const uint4* src = reinterpret_cast<const uint4*>(cache + blk * page_bytes);
  uint4* dst = reinterpret_cast<uint4*>(dense + (base[r] + bi - first[r]) * page_bytes);
  for (int i = threadIdx.x; i < page_bytes / 16; i += blockDim.x) dst[i] = src[i];
}

}  // namespace b200

using namespace b200;

extern "C" {

int b200_latent_prepare(const B200LatentPrep* a, cudaStream_t stream) {
  if (a->T <= 0) return 0;
  if (a->q_rank <= 0 || a->rank <= 0 || a->rot < 0 || (a->rot & 1) || (a->rot && !a->cos_sin) || a->rankp < a->rank ||
      a->rankp + a->rot > a->row || ((a->ldd | a->ldcq | a->kv_col | a->rankp | a->row) & 3))
    return -1;
  const dim3 grid((a->T + 3) / 4);
  return (a->f32 ? launch_pdl(latent_prepare_kernel<float>, grid, dim3(128), 0, stream, *a)
                 : launch_pdl(latent_prepare_kernel<bf16>, grid, dim3(128), 0, stream, *a)) == cudaSuccess ? 0 : -2;
}

int b200_latent_queries(void* q, long long ldq, const void* positions, const float* cos_sin, int H, int qn, int qw, int rot,
                        void* qabs, int rankp, int row, int absorbed, int T, int f32, cudaStream_t stream) {
  if (T <= 0 || rot == 0) return 0;
  if (H <= 0 || (rot & 1) || !cos_sin || (absorbed > 0 && !qabs) || ((ldq | qn | qw | rankp | row) & 3)) return -1;
  const int vec = rot % 8 == 0 ? 4 : 1, n = H * (rot / 2 / vec);
  const int bx = (n + 127) / 128, bz = 16;
  const dim3 grid(bx, (T + bz - 1) / bz, bz);
  if (grid.y > 65535) return -4;
  auto go = [&](auto kernel, auto* tq, auto* ta) {
    return launch_pdl(kernel, grid, dim3(128), 0, stream, tq, ldq, (const int64_t*)positions, cos_sin, H, qn, qw, rot, ta, rankp,
                      row, absorbed, T);
  };
  cudaError_t e;
  if (f32) e = vec == 4 ? go(latent_queries_kernel<float, 4>, (float*)q, (float*)qabs) : go(latent_queries_kernel<float, 1>, (float*)q, (float*)qabs);
  else e = vec == 4 ? go(latent_queries_kernel<bf16, 4>, (bf16*)q, (bf16*)qabs) : go(latent_queries_kernel<bf16, 1>, (bf16*)q, (bf16*)qabs);
  return e == cudaSuccess ? 0 : -2;
}

int b200_latent_gather(const void* cache, const void* block_table, int max_blocks, const void* seq_lens, const void* first,
                       const void* base, int block_size, int row_bytes, void* dense, int num_reqs, int max_pages,
                       cudaStream_t stream) {
  if (num_reqs <= 0 || max_pages <= 0) return 0;
  const long long page = (long long)block_size * row_bytes;
  if (block_size <= 0 || page % 16 || num_reqs > 65535) return -1;
  return launch_pdl(latent_gather_kernel, dim3(max_pages, num_reqs), dim3(128), 0, stream, (const uint8_t*)cache,
                    (const int32_t*)block_table, max_blocks, (const int32_t*)seq_lens, (const int32_t*)first,
                    (const int32_t*)base, block_size, page, (uint8_t*)dense) == cudaSuccess ? 0 : -2;
}

}  // extern "C"
