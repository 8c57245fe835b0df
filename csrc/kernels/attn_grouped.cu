// Grouped-query attention over the pages of attn_bias.cu ([block_size][G * D] keys | [block_size][G * V]
// values): query / key preparation and the decode kernel.
//
//   rotate_kv kernels       rotation and unit norm, or weighted norm and rotation; cache write
//   diff_combine_kernel     difference of a head's two maps, its norm
//   grouped_decode_kernel   bf16, one query row per request: a CTA takes one kv group and one split of the
//                           visible keys, its four warps every fourth tile of 16 keys, each through its own
//                           ring of cp.async stages (no block barrier before the final merge); the group's
//                           query heads are the 16 rows of mma.sync, because the kernel is bound by the cache read
#include "api.h"
#include "sm100.cuh"

namespace b200 {

typedef __nv_bfloat16 bf16;

// ------------------------------------------------------------------- rotation, unit norm, cache write
// Dimension i < rot / 2 of a q or k head is rotated with dimension i + rot / 2, then the head is divided by
// its root mean square over dim (with weights: divided and weighted first, then rotated); v is copied. One warp
// per (token, head).
struct RotateParams {
  const void* qkv;             // [T, ld]: q heads (H * D) | key heads (G * D) | value heads (GV * V); G 0: q only
  long long ld;
  const int64_t* positions;
  const float* cos_sin;        // [positions][cos rot / 2 | sin rot / 2], null: no rotation
  void* q_out;                 // [T, H * D]
  long long ldq;
  const int64_t* slots;
  void* cache;
  int rot, H, G, D, V, dim, block_size, T;
  float eps;
  int GV;
  const float* q_w;            // [D], null: unit norm after the rotation
  const float* k_w;
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
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, heads = p.H + p.G + p.GV;
  const long long x = (long long)blockIdx.x * 4 + warp;
  if (x >= (long long)p.T * heads) return;
  const int t = (int)(x / heads), h = (int)(x % heads);
  const T* row = reinterpret_cast<const T*>(p.qkv) + (size_t)t * p.ld;
  const int64_t slot = h < p.H ? 0 : p.slots[t];
  if (slot < 0) return;
  const int kw = p.G * p.D, vw = p.GV * p.V;
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
  auto inv_rms = [&]() {
    float ss = 0.f;
    for (int i = lane * 4; i < p.D; i += 128) {
      const float4 v = *reinterpret_cast<const float4*>(b + i);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    return 1.f / sqrtf(ss / (float)p.dim + p.eps);
  };
  float inv = 1.f;
  if (p.q_w) {
    const float* w = h < p.H ? p.q_w : p.k_w;
    const float n = inv_rms();
    for (int i = lane * 4; i < p.D; i += 128) {
      const float4 v = *reinterpret_cast<const float4*>(b + i), g = *reinterpret_cast<const float4*>(w + i);
      *reinterpret_cast<float4*>(b + i) = make_float4(v.x * n * g.x, v.y * n * g.y, v.z * n * g.z, v.w * n * g.w);
    }
    __syncwarp();
  }
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
  if (!p.q_w) inv = inv_rms();
  T* dst = h < p.H ? reinterpret_cast<T*>(p.q_out) + (size_t)t * p.ldq + (size_t)h * p.D
                   : page + (int64_t)off * kw + (int64_t)(h - p.H) * p.D;
  for (int i = lane * 4; i < p.D; i += 128) {
    const float4 v = *reinterpret_cast<const float4*>(b + i);
    store4(dst + i, make_float4(v.x * inv, v.y * inv, v.z * inv, v.w * inv));
  }
}

// ---------------------------------------------------------------------------------------------- decode
struct GroupedDecode {
  const bf16* q;
  long long ldq;
  bf16* out;
  long long ldo;
  const bf16* cache;
  const int32_t* block_table;
  const int32_t* seq_lens;
  int max_blocks, H, G, R, D, V, block_size, chunk, splits, window, maps;
  float scale2;                // score scale x log2(e)
  float* tmp_o;                // [B, H, splits, V]
  float* tmp_lse;              // [B, H, splits], log2
  // values inside the key rows: a group's row is ``pitch`` columns, the value its first V, the key those from key_at on
  int pitch, key_at, tied;
  const float* sink;
  float out_scale;
};

static constexpr int kGWarps = 4, kGKeys = 16, kGStages = 3;

__device__ __forceinline__ void g_ldsm4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void g_ldsm4t(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void g_mma(float* d, const uint32_t* a, const uint32_t* b) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ void g_cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void g_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void g_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ float g_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__host__ __device__ inline int g_stage_bytes(int D, int V) { return kGKeys * (D + 8 + V + 8) * 2; }
// (rows of an odd number of 16-byte units)
__host__ __device__ inline int g_tied_row(int pitch) { return (pitch / 8 | 1) * 16; }

// ND, NV: bounds of D / 16 and V / 16.
template <int ND, int NV>
__global__ void __launch_bounds__(kGWarps * 32, ND + NV <= 16 ? 2 : 1) grouped_decode_kernel(GroupedDecode p) {
  extern __shared__ uint4 g_smem[];
  __shared__ float s_m[kGWarps][16], s_l[kGWarps][16];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  // (a group of more than 16 heads takes several CTAs)
  const int b = blockIdx.x, g = blockIdx.y % p.G, head0 = blockIdx.y / p.G * 16, R = min(p.R - head0, 16), split = blockIdx.z;
  const int nd = p.D / 16, nv = p.V / 16, kw = p.G * p.pitch, vw = p.tied ? 0 : p.G * p.V;
  const int ks = p.tied ? g_tied_row(p.pitch) : (p.D + 8) * 2, vs = p.tied ? ks : (p.V + 8) * 2;
  const int stage = p.tied ? kGKeys * ks : g_stage_bytes(p.D, p.V);
  const uint32_t ring = smem_u32(g_smem) + warp * kGStages * stage;
  pdl_wait();
  pdl_launch_dependents();
  const int pos = p.seq_lens[b] - 1, 
            lo = pos <= 0 ? 0 : p.chunk > 0 ? pos / p.chunk * p.chunk : p.window > 0 ? max(pos - p.window + 1, 0) : 0;
  // 16-key tiles of this split: a whole number per warp
  const int first = lo / kGKeys, all = pos < 0 ? 0 : pos / kGKeys + 1 - first;
  const int per = ((all + p.splits - 1) / p.splits + kGWarps - 1) / kGWarps * kGWarps;
  const int ta = first + split * per, tb = min(first + all, ta + per);
  const int n = tb - ta > warp ? (tb - ta - warp + kGWarps - 1) / kGWarps : 0;
  const int32_t* bt = p.block_table + (size_t)b * p.max_blocks;

  // 16-byte unit u of row r of a tile, this lane's first and the step to its next (32 units on)
  const int ku = p.pitch / 8, vu = p.V / 8;
  const int kr0 = lane / ku, ku0 = lane - kr0 * ku, krs = 32 / ku, kus = 32 - krs * ku;
  const int vr0 = lane / vu, vu0 = lane - vr0 * vu, vrs = 32 / vu, vus = 32 - vrs * vu;
  auto load = [&](int i) {                       // tile i of this warp into stage i % kGStages
    if (i < n) {
      const int key = (ta + warp + i * kGWarps) * kGKeys;
      const int page = max(bt[key / p.block_size], 0), off = key % p.block_size;
      const bf16* k = p.cache + (size_t)page * p.block_size * (kw + vw) + (size_t)off * kw + (size_t)g * p.pitch;
      const bf16* v = p.cache + (size_t)page * p.block_size * (kw + vw) + (size_t)p.block_size * kw + (size_t)off * vw + (size_t)g * p.V;
      const uint32_t dst = ring + (i % kGStages) * stage;
      for (int r = kr0, u = ku0; r < kGKeys;) {
        g_cp16(dst + r * ks + u * 16, k + r * kw + u * 8);
        r += krs;
        u += kus;
        if (u >= ku) { u -= ku; ++r; }
      }
      for (int r = p.tied ? kGKeys : vr0, u = vu0; r < kGKeys;) {
        g_cp16(dst + kGKeys * ks + r * vs + u * 16, v + r * vw + u * 8);
        r += vrs;
        u += vus;
        if (u >= vu) { u -= vu; ++r; }
      }
    }
    g_commit();
  };
#pragma unroll
  for (int i = 0; i + 1 < kGStages; ++i) load(i);

  const int r0 = lane >> 2, c0 = (lane & 3) * 2;
  // with maps the query row of a head is zero outside the columns of its own map
  uint32_t qa[ND][4];
  const int dm = p.D / p.maps;
#pragma unroll
  for (int x = 0; x < ND; ++x)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = r0 + (e & 1) * 8, d = x * 16 + c0 + (e >> 1) * 8 - (head0 + r) % p.maps * dm;
      qa[x][e] = r < R && x < nd && d >= 0 && d < dm
                     ? *reinterpret_cast<const uint32_t*>(p.q + (size_t)b * p.ldq + (size_t)(g * p.R + head0 + r) * dm + d) : 0u;
    }
  float o[NV * 2][4];
#pragma unroll
  for (int x = 0; x < NV * 2; ++x) o[x][0] = o[x][1] = o[x][2] = o[x][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  if (p.sink && warp == 0 && split == 0) {       // (counted once; a lane's l is a part of its row's)
    if (r0 < R) { m0 = p.sink[g * p.R + head0 + r0] * 1.4426950408889634f; l0 = (lane & 3) == 0 ? 1.f : 0.f; }
    if (r0 + 8 < R) { m1 = p.sink[g * p.R + head0 + r0 + 8] * 1.4426950408889634f; l1 = (lane & 3) == 0 ? 1.f : 0.f; }
  }
  const uint32_t k_off = ((lane & 7) + ((lane >> 4) << 3)) * ks + ((lane >> 3) & 1) * 16 + p.key_at * 2;
  const uint32_t v_off = (p.tied ? 0 : kGKeys * ks) + (lane & 15) * vs + (lane >> 4) * 16;
  for (int i = 0; i < n; ++i) {
    g_wait<kGStages - 2>();
    __syncwarp();
    load(i + kGStages - 1);                      // (into the stage of the tile before)
    const uint32_t st = ring + (i % kGStages) * stage;
    float s[2][4], z[2][4];                      // (two sums each, to halve the chains of products)
#pragma unroll
    for (int e = 0; e < 4; ++e) s[0][e] = s[1][e] = z[0][e] = z[1][e] = 0.f;
#pragma unroll
    for (int x = 0; x < ND; ++x) {
      if (x < nd) {
        uint32_t kb[4];
        g_ldsm4(kb, st + k_off + x * 32);
        g_mma(x & 1 ? z[0] : s[0], qa[x], kb);
        g_mma(x & 1 ? z[1] : s[1], qa[x], kb + 2);
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) { s[0][e] += z[0][e]; s[1][e] += z[1][e]; }
    const int key = (ta + warp + i * kGWarps) * kGKeys;
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[t][e] *= p.scale2;
    if (key < lo || key + kGKeys - 1 > pos) {
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = key + t * 8 + c0 + e;
          if (j < lo || j > pos) s[t][e] = s[t][e + 2] = -INFINITY;
        }
    }
    float x0 = fmaxf(fmaxf(s[0][0], s[0][1]), fmaxf(s[1][0], s[1][1]));
    float x1 = fmaxf(fmaxf(s[0][2], s[0][3]), fmaxf(s[1][2], s[1][3]));
    x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1));
    x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1));
    x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
    x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
    // the reference maximum is raised lazily, by more than 2^8
    const bool up0 = x0 > m0 + 8.f, up1 = x1 > m1 + 8.f;
    if (__any_sync(0xffffffffu, up0 || up1)) {
      const float a0 = up0 ? (m0 == -INFINITY ? 0.f : g_ex2(m0 - x0)) : 1.f, a1 = up1 ? (m1 == -INFINITY ? 0.f : g_ex2(m1 - x1)) : 1.f;
      if (up0) m0 = x0;
      if (up1) m1 = x1;
      l0 *= a0;
      l1 *= a1;
#pragma unroll
      for (int x = 0; x < NV * 2; ++x) { o[x][0] *= a0; o[x][1] *= a0; o[x][2] *= a1; o[x][3] *= a1; }
    }
#pragma unroll
    for (int t = 0; t < 2; ++t) {
      s[t][0] = g_ex2(s[t][0] - m0); s[t][1] = g_ex2(s[t][1] - m0);
      s[t][2] = g_ex2(s[t][2] - m1); s[t][3] = g_ex2(s[t][3] - m1);
      l0 += s[t][0] + s[t][1];
      l1 += s[t][2] + s[t][3];
    }
    const uint32_t pa[4] = {pack_bf16x2(s[0][0], s[0][1]), pack_bf16x2(s[0][2], s[0][3]), pack_bf16x2(s[1][0], s[1][1]),
                            pack_bf16x2(s[1][2], s[1][3])};
#pragma unroll
    for (int x = 0; x < NV; ++x) {
      if (x < nv) {
        uint32_t vb[4];
        g_ldsm4t(vb, st + v_off + x * 32);
        g_mma(o[2 * x], pa, vb);
        g_mma(o[2 * x + 1], pa, vb + 2);
      }
    }
  }
  g_wait<0>();
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
  l0 += __shfl_xor_sync(0xffffffffu, l0, 2); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  if ((lane & 3) == 0) {
    s_m[warp][r0] = m0; s_m[warp][r0 + 8] = m1;
    s_l[warp][r0] = l0; s_l[warp][r0 + 8] = l1;
  }
  __syncthreads();                               // (every ring is drained: its memory takes the partial sums)
  float* so = reinterpret_cast<float*>(g_smem);  // [warp][16][V]
  float t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
  for (int w = 0; w < kGWarps; ++w) { t0 = fmaxf(t0, s_m[w][r0]); t1 = fmaxf(t1, s_m[w][r0 + 8]); }
  const float f0 = m0 == -INFINITY ? 0.f : g_ex2(m0 - t0), f1 = m1 == -INFINITY ? 0.f : g_ex2(m1 - t1);
#pragma unroll
  for (int x = 0; x < NV * 2; ++x) {
    if (x < 2 * nv) {
      float* d = so + (size_t)(warp * 16 + r0) * p.V + x * 8 + c0;
      *reinterpret_cast<float2*>(d) = make_float2(o[x][0] * f0, o[x][1] * f0);
      *reinterpret_cast<float2*>(d + 8 * p.V) = make_float2(o[x][2] * f1, o[x][3] * f1);
    }
  }
  __syncthreads();
  for (int i = tid; i < R * p.V / 2; i += kGWarps * 32) {
    const int r = i * 2 / p.V, c = i * 2 - r * p.V;
    float mx = -INFINITY, l = 0.f;
#pragma unroll
    for (int w = 0; w < kGWarps; ++w) mx = fmaxf(mx, s_m[w][r]);
    float2 y = make_float2(0.f, 0.f);
#pragma unroll
    for (int w = 0; w < kGWarps; ++w) {
      if (s_m[w][r] != -INFINITY) l += s_l[w][r] * g_ex2(s_m[w][r] - mx);
      const float2 v = *reinterpret_cast<const float2*>(so + (size_t)(w * 16 + r) * p.V + c);
      y.x += v.x;
      y.y += v.y;
    }
    const float inv = l > 0.f ? p.out_scale / l : 0.f;
    const size_t h = (size_t)g * p.R + head0 + r;
    if (p.splits == 1) {
      *reinterpret_cast<uint32_t*>(p.out + (size_t)b * p.ldo + h * p.V + c) = pack_bf16x2(y.x * inv, y.y * inv);
    } else {
      const size_t at = ((size_t)b * p.H + h) * p.splits + split;
      *reinterpret_cast<float2*>(p.tmp_o + at * p.V + c) = make_float2(y.x * inv, y.y * inv);
      if (c == 0) p.tmp_lse[at] = l > 0.f ? mx + log2f(l) : -INFINITY;
    }
  }
}

// Heads of up to 128 values whose half rotation is a multiple of four: a lane holds four values, the partner's
// come by shuffle; a warp takes kRotItems (token, head) pairs, loads first.
static constexpr int kRotItems = 4;
template <typename T>
__global__ void __launch_bounds__(128) rotate_kv_vec_kernel(RotateParams p) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, heads = p.H + p.G + p.GV, c = lane * 4, kw = p.G * p.D, vw = p.GV * p.V;
  const int x0 = (blockIdx.x * 4 + (threadIdx.x >> 5)) * kRotItems, total = p.T * heads;   // (below 2^31: checked)
  int t = x0 / heads, h = x0 - t * heads;
  float4 v[kRotItems], cs[kRotItems], sn[kRotItems];
  T* dst[kRotItems];
  bool turn[kRotItems], is_q[kRotItems];
  const int half = p.rot / 2;
  const bool low = c < half, in_rot = p.cos_sin && c < p.rot;
#pragma unroll
  for (int i = 0; i < kRotItems; ++i) {
    v[i] = cs[i] = sn[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    dst[i] = nullptr;
    turn[i] = h < p.H + p.G;
    is_q[i] = h < p.H;
    if (x0 + i < total) {
      const T* row = reinterpret_cast<const T*>(p.qkv) + (size_t)t * p.ld;
      const int width = turn[i] ? p.D : p.V;
      const int64_t slot = h < p.H ? 0 : p.slots[t];
      if (slot >= 0 && c < width) {
        v[i] = load4<T>(row + (turn[i] ? (size_t)h * p.D : (size_t)(p.H + p.G) * p.D + (size_t)(h - p.H - p.G) * p.V) + c);
        if (h < p.H) {
          dst[i] = reinterpret_cast<T*>(p.q_out) + (size_t)t * p.ldq + (size_t)h * p.D + c;
        } else {
          const uint32_t page = (uint32_t)slot / (uint32_t)p.block_size, off = (uint32_t)slot - page * p.block_size;
          T* base = reinterpret_cast<T*>(p.cache) + page * (p.block_size * (int64_t)(kw + vw));
          dst[i] = turn[i] ? base + off * kw + (int64_t)(h - p.H) * p.D + c
                           : base + (int64_t)p.block_size * kw + off * vw + (int64_t)(h - p.H - p.G) * p.V + c;
        }
        if (turn[i] && in_rot) {
          const float* f = p.cos_sin + (size_t)p.positions[t] * p.rot + (low ? c : c - half);
          cs[i] = *reinterpret_cast<const float4*>(f);
          sn[i] = *reinterpret_cast<const float4*>(f + half);
        }
      }
    }
    if (++h == heads) { h = 0; ++t; }
  }
  auto sum_sq = [](float4 y) {
    float ss = y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w;
#pragma unroll
    for (int k = 16; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
    return ss;
  };
  if (p.q_w) {
    float4 wq = make_float4(0.f, 0.f, 0.f, 0.f), wk = wq;
    if (c < p.D) {
      wq = *reinterpret_cast<const float4*>(p.q_w + c);
      if (p.k_w) wk = *reinterpret_cast<const float4*>(p.k_w + c);
    }
#pragma unroll
    for (int i = 0; i < kRotItems; ++i) {
      const float inv = 1.f / sqrtf(sum_sq(v[i]) / (float)p.dim + p.eps);
      const float4 w = is_q[i] ? wq : wk;
      if (turn[i]) v[i] = make_float4(v[i].x * inv * w.x, v[i].y * inv * w.y, v[i].z * inv * w.z, v[i].w * inv * w.w);
    }
  }
  const int partner = in_rot ? (low ? lane + half / 4 : lane - half / 4) : lane;
#pragma unroll
  for (int i = 0; i < kRotItems; ++i) {
    float4 o;
    o.x = __shfl_sync(0xffffffffu, v[i].x, partner);
    o.y = __shfl_sync(0xffffffffu, v[i].y, partner);
    o.z = __shfl_sync(0xffffffffu, v[i].z, partner);
    o.w = __shfl_sync(0xffffffffu, v[i].w, partner);
    float4 y = v[i];
    if (turn[i] && in_rot) {
      const float g = low ? -1.f : 1.f;
      y = make_float4(y.x * cs[i].x + g * o.x * sn[i].x, y.y * cs[i].y + g * o.y * sn[i].y,
                      y.z * cs[i].z + g * o.z * sn[i].z, y.w * cs[i].w + g * o.w * sn[i].w);
    }
    const float inv = turn[i] && !p.q_w ? 1.f / sqrtf(sum_sq(y) / (float)p.dim + p.eps) : 1.f;
    if (dst[i]) store4(dst[i], make_float4(y.x * inv, y.y * inv, y.z * inv, y.w * inv));
  }
}

// Head sizes that are multiples of 8 (up to 256) whose half rotation is one too: a lane holds eight values, a head
// is a group of LANES lanes. One CTA per token, its warps take the heads in turn, so that a lane needs the
// token's cosines only once. The value row is copied in pieces as wide as a head.
template <typename T> struct Ld8;
template <> struct Ld8<float> {
  static __device__ __forceinline__ void get(const float* p, float* v) {
    *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
    *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(p + 4);
  }
  static __device__ __forceinline__ void put(float* p, const float* v) {
    *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(v);
    *reinterpret_cast<float4*>(p + 4) = *reinterpret_cast<const float4*>(v + 4);
  }
};
template <> struct Ld8<bf16> {
  static __device__ __forceinline__ void get(const bf16* p, float* v) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = unpack_bf16x2(w[i]);
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  }
  static __device__ __forceinline__ void put(bf16* p, const float* v) {
    *reinterpret_cast<uint4*>(p) =
        make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
  }
};

template <typename T, int LANES>
__global__ void __launch_bounds__(128) rotate_kv_row_kernel(RotateParams p) {
  static constexpr int kHeads = 32 / LANES;              // heads of a warp at a time
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = lane % LANES, c = sub * 8;
  const int kw = p.G * p.D, vw = p.GV * p.V, turned = p.H + p.G, heads = turned + (vw + p.D - 1) / p.D;
  const T* row = reinterpret_cast<const T*>(p.qkv) + (size_t)t * p.ld;
  const int64_t slot = p.G ? p.slots[t] : -1;
  T* page = nullptr;
  int off = 0;
  if (slot >= 0) {
    page = reinterpret_cast<T*>(p.cache) + slot / p.block_size * p.block_size * (int64_t)(kw + vw);
    off = (int)(slot % p.block_size);
  }
  const int half = p.rot / 2;
  const bool in = c < p.D, low = c < half, in_rot = p.cos_sin && c < p.rot;
  float cs[8], sn[8], wq[8], wk[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) { cs[i] = 1.f; sn[i] = 0.f; wq[i] = wk[i] = 1.f; }
  if (in_rot) {
    const float* f = p.cos_sin + (size_t)p.positions[t] * p.rot + (low ? c : c - half);
    Ld8<float>::get(f, cs);
    Ld8<float>::get(f + half, sn);
    if (low) {
#pragma unroll
      for (int i = 0; i < 8; ++i) sn[i] = -sn[i];
    }
  }
  if (p.q_w && in) {
    Ld8<float>::get(p.q_w + c, wq);
    if (p.k_w) Ld8<float>::get(p.k_w + c, wk);
  }
  const int partner = in_rot ? (low ? lane + half / 8 : lane - half / 8) : lane;
  auto inv_rms = [&](const float* v) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss = fmaf(v[i], v[i], ss);
#pragma unroll
    for (int k = LANES / 2; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
    return 1.f / sqrtf(ss / (float)p.dim + p.eps);
  };
#pragma unroll 2
  for (int h0 = warp * kHeads; h0 < heads; h0 += 4 * kHeads) {
    const int h = h0 + lane / LANES;
    const bool on = in && h < heads && (h < p.H || page) && (h < turned || (h - turned) * p.D + c < vw);
    float v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = 0.f;
    if (on) Ld8<T>::get(row + (size_t)h * p.D + c, v);
    if (h0 < turned) {                                   // (warp-uniform)
      float inv = 1.f;
      if (p.q_w) {
        inv = inv_rms(v);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] *= h < turned ? inv * (h < p.H ? wq[i] : wk[i]) : 1.f;
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float o = __shfl_sync(0xffffffffu, v[i], partner);
        if (h < turned) v[i] = fmaf(v[i], cs[i], o * sn[i]);
      }
      if (!p.q_w) {
        inv = inv_rms(v);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] *= h < turned ? inv : 1.f;
      }
    }
    if (!on) continue;
    T* dst = h < p.H ? reinterpret_cast<T*>(p.q_out) + (size_t)t * p.ldq + (size_t)h * p.D
             : h < turned ? page + (int64_t)off * kw + (int64_t)(h - p.H) * p.D
                          : page + (int64_t)p.block_size * kw + (int64_t)off * vw + (int64_t)(h - turned) * p.D;
    Ld8<T>::put(dst + c, v);
  }
}

template <typename T>
static int launch_rotate_rows(const RotateParams& p, cudaStream_t stream) {
  const dim3 grid(p.T), block(128);
  cudaError_t e;
  if (p.D <= 16) e = launch_pdl(rotate_kv_row_kernel<T, 2>, grid, block, 0, stream, p);
  else if (p.D <= 32) e = launch_pdl(rotate_kv_row_kernel<T, 4>, grid, block, 0, stream, p);
  else if (p.D <= 64) e = launch_pdl(rotate_kv_row_kernel<T, 8>, grid, block, 0, stream, p);
  else if (p.D <= 128) e = launch_pdl(rotate_kv_row_kernel<T, 16>, grid, block, 0, stream, p);
  else e = launch_pdl(rotate_kv_row_kernel<T, 32>, grid, block, 0, stream, p);
  return e == cudaSuccess ? 0 : -2;
}

bool grouped_decode_fits(const B200BiasAttn* a) {
  if (!a->grouped || a->f32 || a->bias || a->null_entry || a->kw % a->G || a->gate) return false;
  if (a->values_in_keys && (a->maps > 1 || (a->kw / a->G & 7) || (a->key_at & 7))) return false;
  const int D = a->kw / a->G - a->key_at, V = a->vdim;
  return !(D / (a->maps > 1 ? a->maps : 1) & 15) && !(V & 15) && D <= 256 && V <= 256 && a->block_size % kGKeys == 0 &&
         !(((uintptr_t)a->q | (uintptr_t)a->cache) & 15) && !(a->ldq & 7) && !(a->ldo & 1) && a->scale > 0.f;
}

template <int ND, int NV>
static int launch_grouped(const GroupedDecode& p, int rows, cudaStream_t stream) {
  size_t smem = (size_t)kGWarps * kGStages * (p.tied ? kGKeys * g_tied_row(p.pitch) : g_stage_bytes(p.D, p.V));
  const size_t merge = (size_t)kGWarps * 16 * p.V * 4;
  if (smem < merge) smem = merge;
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(grouped_decode_kernel<ND, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  return launch_pdl(grouped_decode_kernel<ND, NV>, dim3(rows, p.G * ((p.R + 15) / 16), p.splits), dim3(kGWarps * 32), smem, stream, p) ==
                 cudaSuccess ? 0 : -2;
}
template <int ND>
static int launch_grouped(const GroupedDecode& p, int rows, cudaStream_t stream) {
  return p.V <= 64 ? launch_grouped<ND, 4>(p, rows, stream) : p.V <= 128 ? launch_grouped<ND, 8>(p, rows, stream)
                                                                          : launch_grouped<ND, 16>(p, rows, stream);
}

int grouped_decode(const B200BiasAttn* a, cudaStream_t stream) {
  GroupedDecode p{(const bf16*)a->q, a->ldq, (bf16*)a->out, a->ldo, (const bf16*)a->cache, (const int32_t*)a->block_table,
                  (const int32_t*)a->seq_lens, a->max_blocks, a->H, a->G, a->H / a->G, a->kw / a->G - a->key_at, a->vdim, a->block_size,
                  a->chunk, a->splits < 1 ? 1 : a->splits, a->window, a->maps > 1 ? a->maps : 1, a->scale * 1.4426950408889634f, (float*)a->tmp_o,
                  (float*)a->tmp_lse, a->kw / a->G, a->key_at, a->values_in_keys, a->sink, a->out_scale};
  if (p.splits > 1 && (!p.tmp_o || !p.tmp_lse)) return -1;
  if ((long)p.G * ((p.R + 15) / 16) > 65535 || p.splits > 65535) return -4;
  const int rc = p.D <= 64 ? launch_grouped<4>(p, a->rows, stream) : p.D <= 128 ? launch_grouped<8>(p, a->rows, stream)
                                                                                : launch_grouped<16>(p, a->rows, stream);
  if (rc || p.splits == 1) return rc;
  return b200_attn_decode_merge(p.tmp_o, p.tmp_lse, p.out, (int)p.ldo, a->rows, p.H, p.V, p.splits, stream);
}

// --------------------------------------------------------- rotation where values are unrotated keys
// One CTA per token. A head of the projection is [first r8 | rest], of which rot are rotated (pairs half of rot apart); the
// query row becomes [rest | first rotated], a group's cache row [first | rest | first rotated]. A thread copies VEC values
// of the rest or turns VEC pairs; the padding after rot is zeros.
struct TiedRotate {
  const void* qk;
  long long ld;
  const int64_t* positions;
  const float* cos_sin;
  void* q_out;
  long long ldq;
  const int64_t* slots;
  void* cache;
  int rot, r8, H, G, D, block_size;
};
template <typename T, int VEC>
__global__ void __launch_bounds__(128) rotate_tied_kernel(TiedRotate p) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, half = p.rot / 2, rest = p.D - p.r8, pitch = p.D + p.r8;
  const int copies = rest / VEC, turns = half / VEC, units = copies + turns, pads = VEC == 1 ? p.r8 - p.rot : 0;
  const T* row = reinterpret_cast<const T*>(p.qk) + (size_t)t * p.ld;
  const int64_t slot = p.slots[t];
  T* line = slot < 0 ? nullptr : reinterpret_cast<T*>(p.cache) + slot * p.G * pitch;   // (pages hold rows only)
  const float* cs = p.cos_sin ? p.cos_sin + (size_t)p.positions[t] * p.rot : nullptr;
  for (int x = threadIdx.x; x < (p.H + p.G) * (units + pads); x += blockDim.x) {
    const int h = x / (units + pads), u = x - h * (units + pads);
    const bool is_q = h < p.H;
    if (!is_q && !line) continue;
    const T* src = row + (size_t)h * p.D;
    T* head = is_q ? reinterpret_cast<T*>(p.q_out) + (size_t)t * p.ldq + (size_t)h * p.D : line + (size_t)(h - p.H) * pitch;
    T* key = is_q ? head : head + p.r8;              // [rest | first rotated]
    if (u < copies) {
      if (VEC == 8) *reinterpret_cast<uint4*>(key + u * 8) = *reinterpret_cast<const uint4*>(src + p.r8 + u * 8);
      else key[u] = src[p.r8 + u];
    } else if (u < units) {
      const int i = (u - copies) * VEC;
      float a[VEC], b[VEC], y[VEC], z[VEC];
      if constexpr (VEC == 8) {
        Ld8<T>::get(src + i, a);
        Ld8<T>::get(src + half + i, b);
      } else {
        a[0] = (float)src[i];
        b[0] = (float)src[half + i];
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const float c = cs[i + e], s = cs[half + i + e];
        y[e] = a[e] * c - b[e] * s;
        z[e] = b[e] * c + a[e] * s;
      }
      T* turned = key + rest;
      if constexpr (VEC == 8) {
        Ld8<T>::put(turned + i, y);
        Ld8<T>::put(turned + half + i, z);
        if (!is_q) {
          Ld8<T>::put(head + i, a);
          Ld8<T>::put(head + half + i, b);
        }
      } else {
        turned[i] = (T)y[0];
        turned[half + i] = (T)z[0];
        if (!is_q) {
          head[i] = src[i];
          head[half + i] = src[half + i];
        }
      }
    } else {
      const int i = p.rot + u - units;
      key[rest + i] = (T)0.f;
      if (!is_q) head[i] = (T)0.f;
    }
  }
}

// ----------------------------------------------------------------------- difference of two maps
// One warp per (token, head): o = first - lam second, over its root mean square over vdim, times scale.
template <typename T>
__global__ void __launch_bounds__(128) diff_combine_kernel(const T* maps, long long ldm, T* out, long long ldo, int H, int V,
                                                           int vdim, long long items, float lam, float eps, float scale) {
  pdl_wait();
  pdl_launch_dependents();
  const long long x = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (x >= items) return;
  const int lane = threadIdx.x & 31, h = (int)(x % H);
  const long long t = x / H;
  const T* src = maps + t * ldm + (size_t)h * 2 * V;
  T* dst = out + t * ldo + (size_t)h * V;
  auto diff = [&](int i) {
    const float4 a = load4<T>(src + i), b = load4<T>(src + V + i);
    return make_float4(a.x - lam * b.x, a.y - lam * b.y, a.z - lam * b.z, a.w - lam * b.w);
  };
  static constexpr int kKeep = 2;                // (groups kept between the passes)
  float4 keep[kKeep];
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < kKeep; ++c) {
    keep[c] = c * 128 + lane * 4 < V ? diff(c * 128 + lane * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    ss += keep[c].x * keep[c].x + keep[c].y * keep[c].y + keep[c].z * keep[c].z + keep[c].w * keep[c].w;
  }
  for (int i = kKeep * 128 + lane * 4; i < V; i += 128) {
    const float4 v = diff(i);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float f = scale / sqrtf(ss / (float)vdim + eps);
#pragma unroll
  for (int c = 0; c < kKeep; ++c)
    if (c * 128 + lane * 4 < V)
      store4(dst + c * 128 + lane * 4, make_float4(keep[c].x * f, keep[c].y * f, keep[c].z * f, keep[c].w * f));
  for (int i = kKeep * 128 + lane * 4; i < V; i += 128) {
    const float4 v = diff(i);
    store4(dst + i, make_float4(v.x * f, v.y * f, v.z * f, v.w * f));
  }
}

}  // namespace b200

using namespace b200;

extern "C" {

int b200_rotate_kv(const void* qkv, long long ld, const void* positions, const void* cos_sin, int rot, float eps,
                   const float* q_w, const float* k_w, void* q_out, long long ldq, const void* slots, void* cache, int H, int G,
                   int GV, int D, int V, int dim, int block_size, int T, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G < 0 || GV < 0 || GV > G || (G && q_w && !k_w) || D <= 0 || (D & 3) || (G && (V <= 0 || (V & 3))) || D > kRotMax || dim <= 0 || dim > D ||
      (cos_sin && ((rot & 1) || rot > dim)) || (ld & 3) || (ldq & 3) || block_size <= 0)
    return -1;
  RotateParams p{qkv, ld, (const int64_t*)positions, (const float*)cos_sin, q_out, ldq, (const int64_t*)slots, cache,
                 rot, H, G, D, V, dim, block_size, T, eps, GV, q_w, k_w};
  const long long items = (long long)T * (H + G + GV);
  const int es = f32 ? 4 : 2;
  const bool aligned = !(((uintptr_t)qkv | (uintptr_t)q_out | (uintptr_t)cache) & 15) && !((ld * es | ldq * es) & 15);
  if (aligned && !(D & 7) && D <= 256 && (!cos_sin || !(rot & 15)) && !(GV * V & 7))
    return f32 ? launch_rotate_rows<float>(p, stream) : launch_rotate_rows<bf16>(p, stream);
  if (D <= 128 && (!G || V <= 128) && (!cos_sin || !(rot & 7)) && items < (1ll << 31) - 64) {
    const dim3 vgrid((unsigned)((items + 4 * kRotItems - 1) / (4 * kRotItems)));
    return (f32 ? launch_pdl(rotate_kv_vec_kernel<float>, vgrid, dim3(128), 0, stream, p)
                : launch_pdl(rotate_kv_vec_kernel<bf16>, vgrid, dim3(128), 0, stream, p)) == cudaSuccess ? 0 : -2;
  }
  const dim3 grid((unsigned)((items + 3) / 4));
  const size_t smem = (size_t)4 * D * 4;
  return (f32 ? launch_pdl(rotate_kv_kernel<float>, grid, dim3(128), smem, stream, p)
              : launch_pdl(rotate_kv_kernel<bf16>, grid, dim3(128), smem, stream, p)) == cudaSuccess ? 0 : -2;
}

int b200_rotate_tied(const void* qk, long long ld, const void* positions, const void* cos_sin, int rot, void* q_out, long long ldq,
                     const void* slots, void* cache, int H, int G, int D, int block_size, int T, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  const int r8 = (rot + 7) / 8 * 8;
  if (H <= 0 || G <= 0 || D <= 0 || rot < 0 || (rot & 1) || r8 > D || (D & 7) || (rot && !cos_sin) || block_size <= 0) return -1;
  const TiedRotate p{qk, ld, (const int64_t*)positions, (const float*)cos_sin, q_out, ldq, (const int64_t*)slots, cache, rot, r8,
                     H, G, D, block_size};
  const int es = f32 ? 4 : 2;
  const bool vec = !(((uintptr_t)qk | (uintptr_t)q_out | (uintptr_t)cache | (uintptr_t)(ld * es) | (uintptr_t)(ldq * es)) & 15) &&
                   !(rot & 15) && !f32;
  cudaError_t e;
  if (vec) e = launch_pdl(rotate_tied_kernel<bf16, 8>, dim3(T), dim3(128), 0, stream, p);
  else if (f32) e = launch_pdl(rotate_tied_kernel<float, 1>, dim3(T), dim3(128), 0, stream, p);
  else e = launch_pdl(rotate_tied_kernel<bf16, 1>, dim3(T), dim3(128), 0, stream, p);
  return e == cudaSuccess ? 0 : -2;
}

int b200_diff_combine(const void* maps, long long ldm, void* out, long long ldo, int H, int V, int vdim, int T, float lam,
                      float eps, float scale, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || V <= 0 || (V & 3) || vdim <= 0 || vdim > V || (ldm & 3) || (ldo & 3)) return -1;
  const long long items = (long long)T * H;
  const dim3 grid((unsigned)((items + 3) / 4));
  return (f32 ? launch_pdl(diff_combine_kernel<float>, grid, dim3(128), 0, stream, (const float*)maps, ldm, (float*)out, ldo, H,
                           V, vdim, items, lam, eps, scale)
              : launch_pdl(diff_combine_kernel<bf16>, grid, dim3(128), 0, stream, (const bf16*)maps, ldm, (bf16*)out, ldo, H, V,
                           vdim, items, lam, eps, scale)) == cudaSuccess ? 0 : -2;
}

}  // extern "C"
