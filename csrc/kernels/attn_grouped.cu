// Grouped-query attention over the pages of attn_bias.cu ([block_size][G * D] keys | [block_size][G * V]
// values): query / key preparation and the decode kernel.
#include "api.h"
#include "sm100.cuh"

namespace b200 {

typedef __nv_bfloat16 bf16;

// ------------------------------------------------------------------- rotation, unit norm, cache write
// Dimension i < rot / 2 of a q or k head is rotated with dimension i + rot / 2, then the head is divided by
// its root mean square over dim; v is copied. One warp per (token, head).
struct RotateParams {
  const void* qkv;             // [T, ld]: q heads (H * D) | key heads (G * D) | value heads (G * V); G 0: q only
  long long ld;
  const int64_t* positions;
  const float* cos_sin;        // [positions][cos rot / 2 | sin rot / 2], null: no rotation
  void* q_out;                 // [T, H * D]
  long long ldq;
  const int64_t* slots;
  void* cache;
  int rot, H, G, D, V, dim, block_size, T;
  float eps;
};

static constexpr int kRotMax = 512;

template <typename T>
__device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<bf16>(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

template <typename T>
__global__ void __launch_bounds__(128) rotate_kv_kernel(RotateParams p) {
  extern __shared__ float rot_smem[];
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, heads = p.H + 2 * p.G;
  const long long x = (long long)blockIdx.x * 4 + warp;
  if (x >= (long long)p.T * heads) return;
  const int t = (int)(x / heads), h = (int)(x % heads);
  const T* row = reinterpret_cast<const T*>(p.qkv) + (size_t)t * p.ld;
  const int64_t slot = h < p.H ? 0 : p.slots[t];
  if (slot < 0) return;
  const int kw = p.G * p.D, vw = p.G * p.V;
  T* page = reinterpret_cast<T*>(p.cache);
  if (h >= p.H) page += slot / p.block_size * p.block_size * (int64_t)(kw + vw);
  const int off = (int)(slot % p.block_size);
  if (h >= p.H + p.G) {
    const int g = h - p.H - p.G;
    const T* src = row + (size_t)(p.H + p.G) * p.D + (size_t)g * p.V;
    T* dst = page + (int64_t)p.block_size * kw + (int64_t)off * vw + (int64_t)g * p.V;
    for (int i = lane * 4; i < p.V; i += 128) store4(dst + i, load4<T>(src + i));
    return;
  }
  float* b = rot_smem + warp * p.D;
  const T* src = row + (size_t)h * p.D;
  for (int i = lane * 4; i < p.D; i += 128) *reinterpret_cast<float4*>(b + i) = load4<T>(src + i);
  __syncwarp();
  const int half = p.rot / 2;
  if (p.cos_sin) {
    const float* cs = p.cos_sin + (size_t)p.positions[t] * p.rot;
    for (int i = lane; i < half; i += 32) {
      const float u = b[i], v = b[i + half], c = cs[i], s = cs[half + i];
      b[i] = u * c - v * s;
      b[i + half] = v * c + u * s;
    }
    __syncwarp();
  }
  float ss = 0.f;
  for (int i = lane * 4; i < p.D; i += 128) {
    const float4 v = *reinterpret_cast<const float4*>(b + i);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float inv = 1.f / sqrtf(ss / (float)p.dim + p.eps);
  T* dst = h < p.H ? reinterpret_cast<T*>(p.q_out) + (size_t)t * p.ldq + (size_t)h * p.D
                   : page + (int64_t)off * kw + (int64_t)(h - p.H) * p.D;
  for (int i = lane * 4; i < p.D; i += 128) {
    const float4 v = *reinterpret_cast<const float4*>(b + i);
    store4(dst + i, make_float4(v.x * inv, v.y * inv, v.z * inv, v.w * inv));
  }
}

bool grouped_decode_fits(const B200BiasAttn* a) { return false; }
int grouped_decode(const B200BiasAttn* a, cudaStream_t stream) { return -4; }

}  // namespace b200

using namespace b200;

extern "C" {

int b200_rotate_kv(const void* qkv, long long ld, const void* positions, const void* cos_sin, int rot, float eps,
                   void* q_out, long long ldq, const void* slots, void* cache, int H, int G, int D, int V, int dim,
                   int block_size, int T, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G < 0 || D <= 0 || (D & 3) || (G && (V <= 0 || (V & 3))) || D > kRotMax || dim <= 0 || dim > D ||
      (cos_sin && ((rot & 1) || rot > dim)) || (ld & 3) || (ldq & 3) || block_size <= 0)
    return -1;
  RotateParams p{qkv, ld, (const int64_t*)positions, (const float*)cos_sin, q_out, ldq, (const int64_t*)slots, cache,
                 rot, H, G, D, V, dim, block_size, T, eps};
  const dim3 grid((unsigned)(((long long)T * (H + 2 * G) + 3) / 4));
  const size_t smem = (size_t)4 * D * 4;
  return (f32 ? launch_pdl(rotate_kv_kernel<float>, grid, dim3(128), smem, stream, p)
              : launch_pdl(rotate_kv_kernel<bf16>, grid, dim3(128), smem, stream, p)) == cudaSuccess ? 0 : -2;
}

}  // extern "C"
