// Attention over a paged cache with separate key and value widths: scores may carry a per-head distance
// bias and a mix of the heads, the softmax a null entry, and a query may be limited to its own chunk or
// window of positions. Grouped heads may come in maps: a group then holds that many keys per token beside one
// value, and head h meets the h % maps-th.
//
//   s[h, i, j] = scale sum_g M[h, g] (q_g(i) . k_g(j)) + bias[h, min(i - j, L - 1)]
//   p[h, i, j] = exp(s) / (null + sum_j exp(s)),   o[h, i] = sum_j p[h, i, j] v_{h / R}(j)
//
// A mix of heads before the softmax is linear in the queries, so it moves to the query side: head h
// gets the query row  q'_h = [ sum_{g in group 0} M[h, g] q_g | sum_{g in group 1} ... ]  over the
// concatenated key heads, one key row per token serves every head (b200_head_mix_kv builds the
// rows and writes the cache), and the score is one dot product of the full key row. Without a mix
// ("grouped") a head's query row meets the columns of its own group only.
//
// Cache of a layer: [num_blocks] pages of  [block_size][kw] keys | [block_size][vw] values,
// kw = key row, vw = value row (all key / value heads), one element type.
//
// Three kernels:
//   bias_attn_any_kernel      any sizes, float or bf16 storage, one CTA per (query row, 4 heads)
//   bias_attn_decode_kernel   bf16, one query row per request: key / value tiles arrive by TMA in two
//                             rings, all heads of a request share them, products on mma.sync (few
//                             query rows per key: the kernel is bound by the cache read), split-KV
//   bias_attn_prefill_kernel  bf16, 128-row query tiles on tcgen05 / TMEM
#include <float.h>

#include <mutex>
#include <unordered_map>

#include "api.h"
#include "sm100.cuh"

namespace b200 {

static constexpr float kLog2e = 1.4426950408889634f;

bool grouped_decode_fits(const B200BiasAttn* a);            // attn_grouped.cu
int grouped_decode(const B200BiasAttn* a, cudaStream_t stream);

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// ------------------------------------------------------------------------- query mix + cache write
struct MixParams {
  const float* qkv;      // [T, ld]: q heads (H * dim) | key heads (G * dim) | value heads (G * vdim)
  long long ld;
  const float* mix;      // [H, H]
  void* q_out;           // [T, H * kw], kw = G * dim
  long long ldq;
  const int64_t* slots;  // [T], < 0: no cache write
  void* cache;
  int H, G, dim, vdim, block_size, T;
};

static constexpr int kMixHeads = 8; // output heads per CTA (blockIdx.y)

// kMixTok: tokens per CTA (each loaded mix coefficient serves that many)
template <typename TO, int kMixTok>
__global__ void __launch_bounds__(256) head_mix_kv_kernel(MixParams p) {
  extern __shared__ float mix_smem[];     // [kMixHeads][H] mix rows, then [kMixTok][H * dim] queries
  pdl_wait();
  pdl_launch_dependents();
  const int t0 = blockIdx.x * kMixTok, h0 = blockIdx.y * kMixHeads;
  const int nt = min(kMixTok, p.T - t0), nh = min(kMixHeads, p.H - h0);
  const int qw = p.H * p.dim, kw = p.G * p.dim, vw = p.G * p.vdim, R = p.H / p.G;
  float* sm = mix_smem;
  float* sq = mix_smem + kMixHeads * p.H;
  for (int i = threadIdx.x; i < kMixHeads * p.H; i += blockDim.x)
    sm[i] = i < nh * p.H ? p.mix[(size_t)h0 * p.H + i] : 0.f;
  for (int t = 0; t < kMixTok; ++t)
    for (int i = threadIdx.x; i < qw; i += blockDim.x)
      sq[t * qw + i] = t < nt ? p.qkv[(size_t)(t0 + t) * p.ld + i] : 0.f;
  __syncthreads();
  TO* qo = reinterpret_cast<TO*>(p.q_out);
  for (int c = threadIdx.x; c < kw; c += blockDim.x) {
    const int g = c / p.dim, d = c - g * p.dim;
    float acc[kMixHeads][kMixTok];
#pragma unroll
    for (int h = 0; h < kMixHeads; ++h)
#pragma unroll
      for (int t = 0; t < kMixTok; ++t) acc[h][t] = 0.f;
    for (int r = 0; r < R; ++r) {
      const int gh = g * R + r;
      float q[kMixTok];
#pragma unroll
      for (int t = 0; t < kMixTok; ++t) q[t] = sq[t * qw + gh * p.dim + d];
#pragma unroll
      for (int h = 0; h < kMixHeads; ++h) {
        const float m = sm[h * p.H + gh];
#pragma unroll
        for (int t = 0; t < kMixTok; ++t) acc[h][t] = fmaf(m, q[t], acc[h][t]);
      }
    }
#pragma unroll
    for (int h = 0; h < kMixHeads; ++h)
#pragma unroll
      for (int t = 0; t < kMixTok; ++t)
        if (h < nh && t < nt) qo[(size_t)(t0 + t) * p.ldq + (size_t)(h0 + h) * kw + c] = from_f<TO>(acc[h][t]);
  }
  if (blockIdx.y == 0) {
    TO* cache = reinterpret_cast<TO*>(p.cache);
    for (int t = 0; t < nt; ++t) {
      const int64_t slot = p.slots[t0 + t];
      if (slot < 0) continue;
      const int64_t blk = slot / p.block_size, off = slot % p.block_size;
      const float* src = p.qkv + (size_t)(t0 + t) * p.ld + qw;
      TO* page = cache + blk * p.block_size * (int64_t)(kw + vw);
      TO* kd = page + off * kw;
      TO* vd = page + (int64_t)p.block_size * kw + off * vw;
      for (int i = threadIdx.x; i < kw; i += blockDim.x) kd[i] = from_f<TO>(src[i]);
      for (int i = threadIdx.x; i < vw; i += blockDim.x) vd[i] = from_f<TO>(src[kw + i]);
    }
  }
}

// Head size a multiple of 4 and RR = heads per group known: a thread takes four consecutive dims of one
// group of one token, holds the RR query values of each in registers and runs over this block's output
// heads; the mix rows lie in shared memory in groups of RR. blockIdx.y: slice of output heads, the last
// slice writes the cache instead.
template <typename TO> struct Store4;
template <> struct Store4<float> {
  static __device__ __forceinline__ void put(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct Store4<__nv_bfloat16> {
  static __device__ __forceinline__ void put(__nv_bfloat16* p, const float* v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  }
};

template <typename TO, int RR>
__global__ void __launch_bounds__(256) head_mix_kv_vec_kernel(MixParams p, int heads_per_block) {
  extern __shared__ float mix_smem[];     // [heads_per_block][H]
  pdl_wait();
  pdl_launch_dependents();
  const int kw = p.G * p.dim, vw = p.G * p.vdim, kw4 = kw / 4, vw4 = vw / 4, d4 = p.dim / 4;
  const size_t stride = (size_t)gridDim.x * blockDim.x, first = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (blockIdx.y + 1 == gridDim.y) {
    TO* cache = reinterpret_cast<TO*>(p.cache);
    const int row4 = kw4 + vw4;
    for (size_t x = first; x < (size_t)p.T * row4; x += stride) {
      const int t = (int)(x / row4), i = (int)(x - (size_t)t * row4);
      const int64_t slot = p.slots[t];
      if (slot < 0) continue;
      const int64_t blk = slot / p.block_size, off = slot % p.block_size;
      TO* page = cache + blk * p.block_size * (int64_t)(kw + vw);
      TO* dst = i < kw4 ? page + off * kw + i * 4 : page + (int64_t)p.block_size * kw + off * vw + (i - kw4) * 4;
      const float4 v = *reinterpret_cast<const float4*>(p.qkv + (size_t)t * p.ld + (size_t)p.H * p.dim + i * 4);
      const float f[4] = {v.x, v.y, v.z, v.w};
      Store4<TO>::put(dst, f);
    }
    return;
  }
  const int h0 = blockIdx.y * heads_per_block, nh = min(heads_per_block, p.H - h0);
  for (int i = threadIdx.x; i < nh * p.H; i += blockDim.x) mix_smem[i] = p.mix[(size_t)h0 * p.H + i];
  __syncthreads();
  for (size_t x = first; x < (size_t)p.T * kw4; x += stride) {
    const int t = (int)(x / kw4), c = (int)(x - (size_t)t * kw4), g = c / d4, d = (c - g * d4) * 4;
    const float* src = p.qkv + (size_t)t * p.ld + (size_t)g * RR * p.dim + d;
    float q[RR][4];
#pragma unroll
    for (int r = 0; r < RR; ++r) {
      const float4 v = *reinterpret_cast<const float4*>(src + r * p.dim);
      q[r][0] = v.x; q[r][1] = v.y; q[r][2] = v.z; q[r][3] = v.w;
    }
    TO* dst = reinterpret_cast<TO*>(p.q_out) + (size_t)t * p.ldq + (size_t)h0 * kw + (size_t)c * 4;
    const float* m = mix_smem + g * RR;
#pragma unroll 2
    for (int h = 0; h < nh; ++h, m += p.H, dst += kw) {
      float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int r = 0; r < RR; ++r) {
        const float w = m[r];
#pragma unroll
        for (int e = 0; e < 4; ++e) a[e] = fmaf(w, q[r][e], a[e]);
      }
      Store4<TO>::put(dst, a);
    }
  }
}

// -------------------------------------------------------------------------------- shared parameters
struct BiasAttnParams {
  const void* q;            // [rows, H * kw]
  long long ldq;
  void* out;                // [rows, H * vdim]
  long long ldo;
  const void* cache;
  const int32_t* block_table;
  int max_blocks;
  const int32_t* seq_lens;
  const int32_t* q_start;   // [num_reqs + 1] first row of each request; null: one row per request
  int num_reqs, rows;
  int H, G, kw, vdim, block_size;
  int qw;                   // width of a head's query row: kw, or kw / G (grouped)
  int chunk;                // > 0: keys of the query's own chunk of this many positions
  float scale;
  const float* bias;        // [H, bias_len] or null
  int bias_len;
  int null_entry;           // softmax counts one entry of score 0 without a value
  // decode
  int splits;
  float* tmp_o;             // [B, H, splits, vdim]
  float* tmp_lse;           // [B, H, splits]
  int mt, hp, ksplit, zslices;
  // prefill
  const int32_t* tile_req;
  const int32_t* tile_q0;
  int k_slots, v_slots, q_stream;
  int* status;
  int window, maps, values_in_keys;
  int own_chunks;           // 64-wide chunks of a query row that meet the head's own key columns
  const void* gate;         // [rows, ldg]
  long long ldg;
  const float* sink;        // [H]: one more entry of the softmax, without a value
  int key_at, pitch, vpitch;   // first key column and columns of a group's key row; columns from value head to value head
  float out_scale;
};

// First position a query at pos sees.
__device__ __forceinline__ int first_key(const BiasAttnParams& p, int pos) {
  return p.chunk > 0 ? pos / p.chunk * p.chunk : p.window > 0 ? max(pos - p.window + 1, 0) : 0;
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

// ------------------------------------------------------------------------------- any-size attention
static constexpr int kAnyKeys = 128;
static constexpr int kAnyAcc = 16;     // outputs per thread: heads * vdim <= 128 * kAnyAcc

template <typename T, int kAnyHeads>
__global__ void __launch_bounds__(128) bias_attn_any_kernel(BiasAttnParams p) {
  extern __shared__ float any_smem[];
  float* sq = any_smem;                                  // [kAnyHeads][qw]
  float* sc = sq + kAnyHeads * p.qw;                     // [kAnyHeads][kAnyKeys]
  __shared__ long long krow[kAnyKeys], vrow[kAnyKeys];
  __shared__ float s_alpha[kAnyHeads], s_l[kAnyHeads];
  pdl_wait();
  pdl_launch_dependents();
  const int row = blockIdx.x, h0 = blockIdx.y * kAnyHeads, nh = min(kAnyHeads, p.H - h0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int vw = p.values_in_keys ? 0 : p.G * p.vdim, R = p.H / p.G;
  int req = row, pos;
  if (p.q_start) {
    int lo = 0, hi = p.num_reqs - 1;                     // last request whose first row is <= row
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (p.q_start[mid] <= row) lo = mid; else hi = mid - 1;
    }
    req = lo;
    pos = p.seq_lens[req] - (p.q_start[req + 1] - row);
  } else {
    pos = p.seq_lens[req] - 1;
  }
  const T* q = reinterpret_cast<const T*>(p.q) + (size_t)row * p.ldq + (size_t)h0 * p.qw;
  for (int i = tid; i < nh * p.qw; i += blockDim.x) sq[i] = to_f(q[i]);
  const T* cache = reinterpret_cast<const T*>(p.cache);
  const int32_t* bt = p.block_table + (size_t)req * p.max_blocks;
  float acc[kAnyAcc];
#pragma unroll
  for (int a = 0; a < kAnyAcc; ++a) acc[a] = 0.f;
  // warp w owns the softmax state of head h0 + w
  float m = p.null_entry ? 0.f : -INFINITY, l = p.null_entry ? 1.f : 0.f;
  if (p.sink && warp < nh) { m = p.sink[h0 + warp]; l = 1.f; }
  for (int base = first_key(p, pos); base <= pos; base += kAnyKeys) {
    const int key = base + tid;
    const bool valid = key <= pos;
    __syncthreads();
    if (valid) {
      const long long page = (long long)bt[key / p.block_size] * p.block_size * (p.kw + vw);
      const int off = key % p.block_size;
      krow[tid] = page + (long long)off * p.kw;
      vrow[tid] = p.values_in_keys ? krow[tid] : page + (long long)p.block_size * p.kw + (long long)off * vw;
      float s[kAnyHeads];
#pragma unroll
      for (int h = 0; h < kAnyHeads; ++h) s[h] = 0.f;
      const T* k = cache + krow[tid];
      if (p.qw < p.kw) {
#pragma unroll
        for (int h = 0; h < kAnyHeads; ++h) {
          if (h >= nh) break;
          const T* kg = k + (size_t)((h0 + h) / R) * p.pitch + p.key_at + (size_t)((h0 + h) % p.maps) * p.qw;
          for (int i = 0; i < p.qw; ++i) s[h] = fmaf(sq[h * p.qw + i], to_f(kg[i]), s[h]);
        }
      } else {
        for (int i = 0; i < p.kw; ++i) {
          const float kv = to_f(k[i]);
#pragma unroll
          for (int h = 0; h < kAnyHeads; ++h) s[h] = fmaf(sq[h * p.kw + i], kv, s[h]);
        }
      }
      for (int h = 0; h < nh; ++h)
        sc[h * kAnyKeys + tid] =
            s[h] * p.scale + (p.bias ? p.bias[(size_t)(h0 + h) * p.bias_len + min(pos - key, p.bias_len - 1)] : 0.f);
    } else {
      for (int h = 0; h < nh; ++h) sc[h * kAnyKeys + tid] = -INFINITY;
    }
    __syncthreads();
    if (warp < nh) {
      float v[kAnyKeys / 32], mx = m;
#pragma unroll
      for (int i = 0; i < kAnyKeys / 32; ++i) {
        v[i] = sc[warp * kAnyKeys + i * 32 + lane];
        mx = fmaxf(mx, v[i]);
      }
      mx = warp_max_f32(mx);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < kAnyKeys / 32; ++i) {
        const float e = expf(v[i] - mx);
        sc[warp * kAnyKeys + i * 32 + lane] = e;
        sum += e;
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      const float a = m == -INFINITY ? 0.f : expf(m - mx);
      l = l * a + sum;
      m = mx;
      if (lane == 0) s_alpha[warp] = a;
    }
    __syncthreads();
    const int nk = min(kAnyKeys, pos + 1 - base);
#pragma unroll
    for (int a = 0; a < kAnyAcc; ++a) {
      const int e = tid + a * 128;
      if (e < nh * p.vdim) {
        const int h = e / p.vdim, d = e - h * p.vdim;
        const T* v = cache + (size_t)((h0 + h) / R) * p.vpitch + d;
        float x = acc[a] * s_alpha[h];
        for (int kk = 0; kk < nk; ++kk) x = fmaf(sc[h * kAnyKeys + kk], to_f(v[vrow[kk]]), x);
        acc[a] = x;
      }
    }
  }
  if (warp < nh && lane == 0) s_l[warp] = l;
  __syncthreads();
  T* o = reinterpret_cast<T*>(p.out) + (size_t)row * p.ldo + (size_t)h0 * p.vdim;
#pragma unroll
  for (int a = 0; a < kAnyAcc; ++a) {
    const int e = tid + a * 128;
    if (e < nh * p.vdim) {
      const float ls = s_l[e / p.vdim];
      float x = ls > 0.f ? acc[a] / ls * p.out_scale : 0.f;
      if (p.gate) x *= sigmoid_f(to_f(reinterpret_cast<const T*>(p.gate)[(size_t)row * p.ldg + h0 + e / p.vdim]));
      o[e] = from_f<T>(x);
    }
  }
}

// ---------------------------------------------------------------------------------- decode (bf16)
__device__ __forceinline__ void ldsm_x4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x2_trans(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];"
               : "=r"(r[0]), "=r"(r[1]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_bf16_16816(float* d, const uint32_t* a, const uint32_t* b) {
  asm(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

static constexpr int kDecWarps = 8;      // 255 registers each
static constexpr int kDecThreads = kDecWarps * 32;
static constexpr int kDecMaxSlots = 4;

struct DecodeSmem {                      // byte offsets; the rings are 1024-byte aligned
  int k, v, q, s, p, stat, bars, total;
};
__host__ __device__ inline DecodeSmem decode_smem(int tk, int hp, int nkc, int nvc, int prow, int ksplit, int k_slots,
                                                  int v_slots, bool q_smem) {
  DecodeSmem d;
  int o = 0;
  d.k = o; o += k_slots * nkc * tk * 128;
  d.v = o; o += v_slots * nvc * tk * 128;
  d.q = o; o += q_smem ? hp * (nkc * 64 + 8) * 2 : 0;
  d.s = o; o += 2 * ksplit * hp * (tk + 8) * 4;
  o = (o + 15) & ~15;
  d.p = o; o += 2 * prow * (tk + 8) * 2;
  d.stat = o; o += 3 * hp * 4;
  o = (o + 15) & ~15;
  d.bars = o; o += 2 * kDecMaxSlots * 8;
  d.total = o;
  return d;
}

// grid (request, split, slice of the kv groups). TK keys per tile; MAXI: 16 x 8 output tiles a warp keeps in registers; CPW:
// 64-wide chunks of the query rows it keeps there (0: the queries stay in shared memory); HPW: heads per
// warp in the softmax. (Shared memory leaves next to no L1 cache: nothing may spill.) Key and value
// rows arrive by TMA in 128-byte swizzled chunks of 64 columns. Three tiles are in work at a time, with
// one barrier per round: the scores of tile t + 1 (each warp a slice of the key row, partial sums in
// shared memory), the softmax of tile t, the output product of tile t - 1.
template <int TK, int MAXI, int CPW, int HPW>
__global__ void __launch_bounds__(kDecThreads, 1)
    bias_attn_decode_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                            BiasAttnParams p) {
  extern __shared__ uint8_t dec_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(dec_raw) + 1023) & ~uintptr_t(1023));
  // this CTA's heads: the groups of its z slice
  const int G = p.G / gridDim.z, H = p.H / gridDim.z, h_base = blockIdx.z * H, v_col = blockIdx.z * G * p.vdim;
  const int nkc = (p.kw + 63) / 64, nvc = (G * p.vdim + 63) / 64, prow = G * p.mt * 16;
  const DecodeSmem L = decode_smem(TK, p.hp, nkc, nvc, prow, p.ksplit, p.k_slots, p.v_slots, CPW == 0);
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem + L.q);
  float* sS = reinterpret_cast<float*>(smem + L.s);
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(smem + L.p);
  float* s_alpha = reinterpret_cast<float*>(smem + L.stat);
  float* s_l = s_alpha + 2 * p.hp;
  uint64_t* k_full = reinterpret_cast<uint64_t*>(smem + L.bars);
  uint64_t* v_full = k_full + kDecMaxSlots;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = blockIdx.x, split = blockIdx.y;
  const int R = H / G, ps = TK + 8, ss = TK + 8, s_buf = p.ksplit * p.hp * ss, p_buf = prow * ps;
  const int k_slot_bytes = nkc * TK * 128, v_slot_bytes = nvc * TK * 128;

  // what a product may read and nothing fills has to be finite
  for (int i = tid; i < 2 * p_buf / 8; i += kDecThreads) reinterpret_cast<uint4*>(sP)[i] = make_uint4(0, 0, 0, 0);
  if (tid == 0) {
    for (int i = 0; i < kDecMaxSlots; ++i) {
      mbar_init(&k_full[i], kDecWarps);
      mbar_init(&v_full[i], kDecWarps);
    }
    mbar_fence_init();
  }
  pdl_wait();
  pdl_launch_dependents();
  const int seq_len = p.seq_lens[b], pos = seq_len - 1;
  int chunk = (seq_len + p.splits - 1) / p.splits;
  chunk = (chunk + TK - 1) / TK * TK;
  const int t0 = split * chunk, t1 = min(seq_len, t0 + chunk);
  const int ntiles = t1 > t0 ? (t1 - t0 + TK - 1) / TK : 0;
  __syncthreads();

  // Every warp fetches its share of a tile's 64-wide chunks (one copy per chunk and page part of rpl
  // rows; lane l looks up the page of part l, lane 0 issues). In a slot: [part][chunk][rpl rows][64]. A
  // slot is free once the round that used it has passed its barrier.
  const int rpl = min(p.block_size, TK), loads = TK / rpl;
  const int32_t* bt = p.block_table + (size_t)b * p.max_blocks;
  const int nblk = (seq_len + p.block_size - 1) / p.block_size;
  auto page_of = [&](int t) {
    const int bi = (t0 + t * TK + lane * rpl) / p.block_size;
    return max(t < ntiles && lane < loads && bi < nblk ? bt[bi] : 0, 0);
  };
  auto load = [&](const CUtensorMap* map, uint64_t* bar, int ring, int chunks, int col, int first, int t, int blk) {
    const int row = p.block_size > TK ? (t0 + t * TK) % p.block_size : 0;
    const int n = first < chunks ? (chunks - first + kDecWarps - 1) / kDecWarps : 0;
    if (lane == 0) mbar_expect_tx(bar, n * TK * 128);
    for (int l = 0; l < loads; ++l) {
      const int page = __shfl_sync(0xffffffffu, blk, l);
      if (lane == 0)
        for (int c = first; c < chunks; c += kDecWarps)
          tma_load_3d(smem + ring + (l * chunks + c) * rpl * 128, map, bar, col + c * 64, row, page);
    }
  };
  const int v_first = (warp + kDecWarps - nkc % kDecWarps) % kDecWarps;   // value chunks go on where the key chunks end
  if (ntiles > 0) {
    if (tid == 0) { tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV); }
    for (int i = 0; i < min(p.k_slots, ntiles); ++i)
      load(&tmK, &k_full[i], L.k + i * k_slot_bytes, nkc, 0, warp, i, page_of(i));
    for (int i = 0; i < min(p.v_slots, ntiles); ++i)
      load(&tmV, &v_full[i], L.v + i * v_slot_bytes, nvc, v_col, v_first, i, page_of(i));
  }
  // pages of the next tile of each ring, looked up one round ahead
  int k_page = page_of(p.k_slots), v_page = page_of(p.v_slots);
  // scores: this warp's 16 heads, slice of the key row (chunks c0 ..) and 8-key columns npart, npart + nsplit ..
  constexpr int kNT = TK / 8;
  const int mtiles = p.hp / 16, cper = (nkc + p.ksplit - 1) / p.ksplit;
  const int mtile = warp % mtiles, kpart = (warp / mtiles) % p.ksplit, npart = warp / (mtiles * p.ksplit);
  int nsplit = 1;                          // a power of two
  while (2 * nsplit <= kNT && 2 * nsplit * mtiles * p.ksplit <= kDecWarps) nsplit *= 2;
  const int c0 = kpart * cper, nc = npart < nsplit ? min(cper, nkc - c0) : 0;
  const int qs = nkc * 64 + 8;
  uint32_t qa[CPW > 0 ? CPW : 1][4][4];
  {
    const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.q) + (size_t)b * p.ldq + (size_t)h_base * p.kw;
    if (CPW == 0) {
      for (int h = warp; h < p.hp; h += kDecWarps)
        for (int i = lane; i < qs / 8; i += 32)
          *reinterpret_cast<uint4*>(sQ + h * qs + i * 8) =
              h < H && i * 8 < p.kw ? *reinterpret_cast<const uint4*>(q + (size_t)h * p.kw + i * 8) : make_uint4(0, 0, 0, 0);
      __syncthreads();
    } else {
#pragma unroll
      for (int c = 0; c < CPW; ++c)
#pragma unroll
        for (int kk = 0; kk < 4; ++kk)
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const int h = mtile * 16 + (lane >> 2) + (x & 1) * 8, k = (c0 + c) * 64 + kk * 16 + (lane & 3) * 2 + (x >> 1) * 8;
            qa[c][kk][x] = h < H && c < nc && k < p.kw ? *reinterpret_cast<const uint32_t*>(q + (size_t)h * p.kw + k) : 0u;
          }
    }
  }
  const uint32_t q_addr = smem_u32(sQ + (mtile * 16 + (lane & 15)) * qs + (lane >> 4) * 8) + c0 * 128;
  const uint32_t k_off = c0 * rpl * 128 + (lane & 7) * 128;
  uint32_t n_off[kNT];                     // where the 8 keys of a column start in a slot
#pragma unroll
  for (int n = 0; n < kNT; ++n) n_off[n] = n * 8 / rpl * (nkc * rpl * 128) + n * 8 % rpl * 128;
  const uint32_t u0 = ((lane >> 3) ^ (lane & 7)) << 4, u1 = ((4 + (lane >> 3)) ^ (lane & 7)) << 4;
  float* s_dst = sS + (size_t)(kpart * p.hp + mtile * 16 + (lane >> 2)) * ss + (lane & 3) * 2;
  // outputs: consecutive 8-column pieces in (group, 16-head tile, column) order
  const int n_vt = p.vdim / 8, items = G * p.mt * n_vt, per_warp = (items + kDecWarps - 1) / kDecWarps;
  const int i0 = warp * per_warp, cnt = max(0, min(items - i0, per_warp)), gm0 = i0 / n_vt, nt0 = i0 - gm0 * n_vt;
  const bool one_tile = nt0 + cnt <= n_vt;
  const int g0 = gm0 / p.mt, mi0 = gm0 - g0 * p.mt, v_row = lane & (TK - 1);
  float o[MAXI][4];
#pragma unroll
  for (int i = 0; i < MAXI; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  // softmax state of heads warp, warp + 8, ...: the maximum (log2 domain) is uniform, the sum per lane
  const bool counts_null = p.null_entry && split == 0;
  const int last = p.bias_len - 1;
  float m[HPW], l[HPW], far[HPW];
  int p_off[HPW];
#pragma unroll
  for (int i = 0; i < HPW; ++i) {
    const int h = min(warp + i * kDecWarps, H - 1), g = h / R;
    m[i] = counts_null ? 0.f : -INFINITY;
    l[i] = counts_null && lane == 0 ? 1.f : 0.f;
    far[i] = p.bias ? p.bias[(size_t)(h_base + h) * p.bias_len + last] * kLog2e : 0.f;
    p_off[i] = (g * p.mt * 16 + h - g * R) * ps + lane;
  }
  const uint32_t v_off = v_row / rpl * (nvc * rpl * 128) + v_row % rpl * 128;
  const uint32_t k_base = smem_u32(smem + L.k), v_base = smem_u32(smem + L.v);
  int ksl = 0, vsl = 0, k_free = 0, v_free = 0;
  uint32_t kph = 0, vph = 0;
  bool ok = true;       // after a wait that ran out the warp goes on without waiting (barriers stay matched)

  for (int t = -1; t <= ntiles && ntiles > 0; ++t) {
    // the last round used key tile t and value tile t - 2
    if (t >= 0 && t + p.k_slots < ntiles) {
      load(&tmK, &k_full[k_free], L.k + k_free * k_slot_bytes, nkc, 0, warp, t + p.k_slots, k_page);
      k_page = page_of(t + 1 + p.k_slots);
      if (++k_free == p.k_slots) k_free = 0;
    }
    if (t >= 2 && t - 2 + p.v_slots < ntiles) {
      load(&tmV, &v_full[v_free], L.v + v_free * v_slot_bytes, nvc, v_col, v_first, t - 2 + p.v_slots, v_page);
      v_page = page_of(t - 1 + p.v_slots);
      if (++v_free == p.v_slots) v_free = 0;
    }
    // bias of this round's softmax, asked for before the scores
    const bool near = p.bias && pos - (t0 + t * TK + TK - 1) < last;
    float bias[HPW];
#pragma unroll
    for (int i = 0; i < HPW; ++i) {
      bias[i] = far[i];
      if (near && t >= 0 && warp + i * kDecWarps < H)
        bias[i] = __ldg(p.bias + (size_t)(h_base + warp + i * kDecWarps) * p.bias_len + min(max(pos - t0 - t * TK - lane, 0), last)) * kLog2e;
    }
    if (t + 1 < ntiles) {
      // ---- scores of tile t + 1
      ok = ok && __all_sync(0xffffffffu, mbar_wait(&k_full[ksl], kph, p.status));
      const uint32_t ka = k_base + ksl * k_slot_bytes + k_off;
      float* sd = s_dst + ((t + 1) & 1) * s_buf;
      if (nc > 0) {
        float d[kNT][4];
#pragma unroll
        for (int n = 0; n < kNT; ++n) d[n][0] = d[n][1] = d[n][2] = d[n][3] = 0.f;
        auto chunk_products = [&](int c, const uint32_t (&a)[4][4]) {
#pragma unroll
          for (int n = 0; n < kNT; ++n) {
            if ((n & (nsplit - 1)) != npart) continue;
            uint32_t kb[8];
            ldsm_x4(kb, ka + c * rpl * 128 + n_off[n] + u0);
            ldsm_x4(kb + 4, ka + c * rpl * 128 + n_off[n] + u1);
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) mma_bf16_16816(d[n], a[kk], kb + 2 * kk);
          }
        };
        if (CPW == 0) {
          for (int c = 0; c < nc; ++c) {
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) ldsm_x4(qa[0][kk], q_addr + c * 128 + kk * 32);
            chunk_products(c, qa[0]);
          }
        } else {
#pragma unroll
          for (int c = 0; c < CPW; ++c)
            if (c < nc) chunk_products(c, qa[c]);
        }
#pragma unroll
        for (int n = 0; n < kNT; ++n) {
          if ((n & (nsplit - 1)) != npart) continue;
          *reinterpret_cast<float2*>(sd + n * 8) = make_float2(d[n][0], d[n][1]);
          *reinterpret_cast<float2*>(sd + 8 * ss + n * 8) = make_float2(d[n][2], d[n][3]);
        }
      }
      if (++ksl == p.k_slots) { ksl = 0; kph ^= 1; }
    }
    if (t >= 0 && t < ntiles) {
      // ---- softmax of tile t: one key per lane
      const int tok0 = t0 + t * TK;
      const bool mine = lane < TK && tok0 + lane < t1;
      const float* ssrc = sS + (t & 1) * s_buf + (lane & (TK - 1));
      __nv_bfloat16* pd = sP + (t & 1) * p_buf;
      float x[HPW];
#pragma unroll
      for (int i = 0; i < HPW; ++i) x[i] = warp + i * kDecWarps < H ? ssrc[(warp + i * kDecWarps) * ss] : 0.f;
      for (int k = 1; k < p.ksplit; ++k) {
#pragma unroll
        for (int i = 0; i < HPW; ++i)
          if (warp + i * kDecWarps < H) x[i] += ssrc[(k * p.hp + warp + i * kDecWarps) * ss];
      }
#pragma unroll
      for (int i = 0; i < HPW; ++i) {
        const int h = warp + i * kDecWarps;
        if (h < H) {
          x[i] = mine ? fmaf(x[i], kLog2e, bias[i]) : -INFINITY;
          const float mn = fmaxf(m[i], warp_max_f32(x[i])), e = ex2_approx(x[i] - mn);
          const float a = m[i] == -INFINITY ? 0.f : ex2_approx(m[i] - mn);
          m[i] = mn;
          l[i] = fmaf(l[i], a, e);
          if (lane < TK) pd[p_off[i]] = __float2bfloat16(e);
          if (lane == 0) s_alpha[(t & 1) * p.hp + h] = a;
        }
      }
    }
    if (t >= 1) {
      // ---- output product of tile t - 1
      ok = ok && __all_sync(0xffffffffu, mbar_wait(&v_full[vsl], vph, p.status));
      const __nv_bfloat16* pp = sP + ((t - 1) & 1) * p_buf + (size_t)(lane & 15) * ps + (lane >> 4) * 8;
      const float* al = s_alpha + ((t - 1) & 1) * p.hp;
      const uint32_t va = v_base + vsl * v_slot_bytes + v_off;
      uint32_t pa[TK / 16][4];
      float al0 = 0.f, al1 = 0.f;
      int gm = gm0, nt = nt0, g = g0, mi = mi0, u = (g0 * p.vdim >> 3) + nt0;   // u: 16-byte unit of the value row
      if (cnt > 0 && one_tile) {      // (a warp without pieces has no place in P either)
        // every piece belongs to the same 16 heads: all loads first
#pragma unroll
        for (int kk = 0; kk < TK / 16; ++kk) ldsm_x4(pa[kk], smem_u32(pp + gm * 16 * ps + kk * 16));
        const int r0 = mi * 16 + (lane >> 2);
        al0 = r0 < R ? al[g * R + r0] : 0.f;
        al1 = r0 + 8 < R ? al[g * R + r0 + 8] : 0.f;
#pragma unroll
        for (int i4 = 0; i4 < MAXI; i4 += 4) {
          uint32_t vb[4][4];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int uu = u + i4 + i;
            const uint32_t addr = va + (uu >> 3) * (rpl * 128) + (((uu & 7) ^ (v_row & 7)) << 4);
            if (i4 + i < cnt) { if (TK == 32) ldsm_x4_trans(vb[i], addr); else ldsm_x2_trans(vb[i], addr); }
          }
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if (i4 + i < cnt) {
              float* d = o[i4 + i];
              d[0] *= al0; d[1] *= al0; d[2] *= al1; d[3] *= al1;
#pragma unroll
              for (int kk = 0; kk < TK / 16; ++kk) mma_bf16_16816(d, pa[kk], vb[i] + 2 * kk);
            }
          }
        }
      } else {
        bool fresh = true;
#pragma unroll
      for (int i = 0; i < MAXI; ++i) {
        if (i < cnt) {
          uint32_t vb[4];
          const uint32_t addr = va + (u >> 3) * (rpl * 128) + (((u & 7) ^ (v_row & 7)) << 4);
          if (TK == 32) ldsm_x4_trans(vb, addr); else ldsm_x2_trans(vb, addr);
          if (fresh) {
#pragma unroll
            for (int kk = 0; kk < TK / 16; ++kk) ldsm_x4(pa[kk], smem_u32(pp + gm * 16 * ps + kk * 16));
            const int r0 = mi * 16 + (lane >> 2);
            al0 = r0 < R ? al[g * R + r0] : 0.f;
            al1 = r0 + 8 < R ? al[g * R + r0 + 8] : 0.f;
          }
          o[i][0] *= al0; o[i][1] *= al0; o[i][2] *= al1; o[i][3] *= al1;
#pragma unroll
          for (int kk = 0; kk < TK / 16; ++kk) mma_bf16_16816(o[i], pa[kk], vb + 2 * kk);
          ++u;
          fresh = ++nt == n_vt;
          if (fresh) {
            nt = 0;
            ++gm;
            if (++mi == p.mt) { mi = 0; ++g; } else { u -= n_vt; }
          }
        }
      }
      }
      if (++vsl == p.v_slots) { vsl = 0; vph ^= 1; }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < HPW; ++i) {
    const int h = warp + i * kDecWarps;
    if (h < H) {
#pragma unroll
      for (int k2 = 16; k2 > 0; k2 >>= 1) l[i] += __shfl_xor_sync(0xffffffffu, l[i], k2);
      if (lane == 0) {
        s_l[h] = l[i];
        if (p.splits > 1) p.tmp_lse[((size_t)b * p.H + h_base + h) * p.splits + split] = l[i] > 0.f ? m[i] + log2f(l[i]) : -INFINITY;
      }
    }
  }
  __syncthreads();
  if (!ok) return;
  int nt = nt0, g = g0, mi = mi0;
#pragma unroll
  for (int i = 0; i < MAXI; ++i) {
    if (i < cnt) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = mi * 16 + (lane >> 2) + half * 8;
        if (r < R) {
          const int h = g * R + r, d = nt * 8 + (lane & 3) * 2;
          const float inv = s_l[h] > 0.f ? 1.f / s_l[h] : 0.f;
          const float x0 = o[i][half * 2] * inv, x1 = o[i][half * 2 + 1] * inv;
          if (p.splits == 1) {
            *reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)b * p.ldo +
                                         (size_t)(h_base + h) * p.vdim + d) = pack_bf16x2(x0, x1);
          } else {
            float* t = p.tmp_o + (((size_t)b * p.H + h_base + h) * p.splits + split) * p.vdim + d;
            t[0] = x0;
            t[1] = x1;
          }
        }
      }
      if (++nt == n_vt) {
        nt = 0;
        if (++mi == p.mt) { mi = 0; ++g; }
      }
    }
  }
}

// --------------------------------------------------------------------------------- prefill (bf16)
// One CTA = one 128-row query tile of one request and one head, key tiles of 128. The query row of a
// head is as wide as all key heads together (kw), so the score product is cut into 64-wide chunks that
// arrive in a ring; the query tile stays in shared memory when it fits (else its chunks ride in the
// ring beside the keys'). S is double-buffered in TMEM, P goes back to TMEM as bf16 and is the A operand
// of P V, O accumulates in TMEM (lazy reference maximum, in-place rescale).
// Warps: 0 TMA producer, 1 MMA issuer + TMEM owner, 2..9 softmax, two threads per query row (64 keys
// each) that exchange their row maximum through shared memory.
// The bias of a warp's 32 rows and 128 keys depends on 159 distances only: the pair of warps keeps
// that window of the table in shared memory, filled one tile ahead.
static constexpr int kBQ = 128, kBKeys = 128, kChunkBytes = 128 * 128;   // chunk: 128 rows x 64 bf16
static constexpr int kMaxKSlots = 8, kMinKSlots = 3, kWin = 160;
static constexpr int kPrefillThreads = 320;

struct alignas(8) BiasPrefillBars {
  uint64_t q_full, k_full[kMaxKSlots], k_empty[kMaxKSlots], v_full[2], v_empty[2];
  uint64_t s_full[2], s_empty[2], p_full[2], p_empty[2], o_full;
  uint32_t tmem_base;
  float row_max[2][2][kBQ];          // [tile parity][half][row]
  float window[2][4][kWin];          // [tile parity][quarter]: log2-domain bias by distance
};

__device__ __forceinline__ void pair_sync(int quarter) {             // the two warps of a row quarter
  asm volatile("bar.sync %0, 64;" ::"r"(quarter + 1) : "memory");
}

__global__ void __launch_bounds__(kPrefillThreads, 1)
    bias_attn_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                             const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmS,
                             BiasAttnParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nkc = (p.qw + 63) / 64, nvc = (p.vdim + 63) / 64;
  const int slot_bytes = p.q_stream ? 2 * kChunkBytes : kChunkBytes;      // [keys | queries]
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + (p.q_stream ? 0 : nkc * kChunkBytes);
  uint8_t* sV = sK + p.k_slots * slot_bytes;
  BiasPrefillBars* bars = reinterpret_cast<BiasPrefillBars*>(sV + p.v_slots * nvc * kChunkBytes);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // late tiles of a prompt see the most keys: they go first, so that the last CTAs to run are short
  const int tile = gridDim.x - 1 - blockIdx.x, h = blockIdx.y, hkv = h / (p.H / p.G);
  const int req = p.tile_req[tile], q0 = p.tile_q0[tile];
  const int q_begin = p.q_start[req], q_len = p.q_start[req + 1] - q_begin;
  const int seq_len = p.seq_lens[req], ctx_off = seq_len - q_len;
  const int rows = min(kBQ, q_len - q0);
  // first key tile: that of the first row's first key
  const int lo_tile = first_key(p, ctx_off + q0) / kBKeys;
  const int ntiles = (ctx_off + q0 + rows - 1) / kBKeys + 1 - lo_tile;
  const int k_col = p.own_chunks < nkc ? hkv * p.pitch : p.qw < p.kw ? hkv * p.pitch + p.key_at + h % p.maps * p.qw : 0;
  // TMEM columns: S buffers (128 each), then O, then two P buffers (64 each)
  const int s_bufs = p.vdim > 128 ? 1 : 2;
  const int o_cols = p.vdim > 128 ? 256 : 128;

  if (threadIdx.x == 0) {
    mbar_init(&bars->q_full, 1);
    for (int i = 0; i < p.k_slots; ++i) { mbar_init(&bars->k_full[i], 1); mbar_init(&bars->k_empty[i], 1); }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars->v_full[i], 1);
      mbar_init(&bars->v_empty[i], 1);
      mbar_init(&bars->s_full[i], 1);
      mbar_init(&bars->s_empty[i], 8);
      mbar_init(&bars->p_full[i], 8);
      mbar_init(&bars->p_empty[i], 1);
    }
    mbar_init(&bars->o_full, 1);
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(&bars->tmem_base, 512); tmem_relinquish(); }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_s = bars->tmem_base, tmem_o = tmem_s + s_bufs * kBKeys, tmem_p = tmem_o + o_cols;

  if (warp == 0) {
    // A 128-key tile spans up to 16 pages; lane l looks up and fetches the l-th one, so that the
    // look-ups of a tile run side by side.
    const int rpl = min(p.block_size, kBKeys), loads = kBKeys / rpl;
    const int32_t* bt = p.block_table + (size_t)req * p.max_blocks;
    const int nblk = (seq_len + p.block_size - 1) / p.block_size;
    auto page_of = [&](int j) {
      const int bi = ((lo_tile + j) * kBKeys + lane * rpl) / p.block_size;
      return max(lane < loads && bi < nblk ? bt[bi] : bt[0], 0);
    };
    if (lane == 0) {
      tma_prefetch_desc(&tmQ);
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmV);
      if (!p.q_stream) {
        mbar_expect_tx(&bars->q_full, nkc * kChunkBytes);
        for (int c = 0; c < nkc; ++c)
          tma_load_2d(sQ + c * kChunkBytes, &tmQ, &bars->q_full, h * p.qw + c * 64, q_begin + q0);
      }
    }
    int sl = 0, blk = page_of(0), blk_prev = 0;
    uint32_t ph = 1;
    bool ok = true;
    // Order K0 K1 V0 K2 V1 ... K(n-1) V(n-2) V(n-1): the order in which the MMA warp consumes them.
    for (int j = 0; j <= ntiles && ok; ++j) {
      const int next = j + 1 < ntiles ? page_of(j + 1) : 0;
      if (j < ntiles) {
        const int row = p.block_size > kBKeys ? ((lo_tile + j) * kBKeys) % p.block_size : 0;
        for (int c = 0; c < nkc; ++c) {
          ok = __all_sync(0xffffffffu, mbar_wait(&bars->k_empty[sl], ph, p.status));
          if (!ok) break;
          uint8_t* dst = sK + sl * slot_bytes;
          if (lane == 0) {
            mbar_expect_tx(&bars->k_full[sl], slot_bytes);
            if (p.q_stream)
              tma_load_2d(dst + kChunkBytes, &tmQ, &bars->k_full[sl], h * p.qw + c * 64, q_begin + q0);
          }
          __syncwarp();
          if (lane < loads) {
            const bool own = c < p.own_chunks;
            tma_load_3d(dst + lane * rpl * 128, own ? &tmK : &tmS, &bars->k_full[sl],
                        own ? k_col + c * 64 : (c - p.own_chunks) * 64, row, blk);
          }
          if (++sl == p.k_slots) { sl = 0; ph ^= 1; }
        }
      }
      if (j >= 1 && ok) {
        const int i = j - 1, vs = i % p.v_slots;
        const int row = p.block_size > kBKeys ? ((lo_tile + i) * kBKeys) % p.block_size : 0;
        ok = __all_sync(0xffffffffu, mbar_wait(&bars->v_empty[vs], ((i / p.v_slots) & 1) ^ 1, p.status));
        if (!ok) break;
        if (lane == 0) mbar_expect_tx(&bars->v_full[vs], nvc * kChunkBytes);
        __syncwarp();
        if (lane < loads)
          for (int c = 0; c < nvc; ++c)
            tma_load_3d(sV + (vs * nvc + c) * kChunkBytes + lane * rpl * 128, &tmV, &bars->v_full[vs],
                        hkv * p.vpitch + c * 64, row, blk_prev);
      }
      blk_prev = blk;
      blk = next;
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_qk = umma_idesc_bf16(kBQ, kBKeys, 0, 0);
      const uint32_t idesc_pv = umma_idesc_bf16(kBQ, (p.vdim + 15) & ~15, 0, 1);
      bool ok = p.q_stream || mbar_wait(&bars->q_full, 0, p.status);
      // descriptors advance by plain adds: 16 k elements are 32 bytes = 2 address units
      const uint64_t qd0 = umma_desc_k_sw128(smem_u32(sQ), 1024), kd0 = umma_desc_k_sw128(smem_u32(sK), 1024);
      const uint64_t vd0 = umma_desc_mn_sw128(smem_u32(sV), kChunkBytes, 1024);
      const int tail = (p.qw - (nkc - 1) * 64 + 15) / 16;          // instructions of the last chunk
      int ksl = 0;
      uint32_t kph = 0;
      for (int j = 0; j <= ntiles && ok; ++j) {
        if (j < ntiles) {
          const int sb = j % s_bufs;
          const uint32_t d = tmem_s + sb * kBKeys;
          if (!mbar_wait(&bars->s_empty[sb], ((j / s_bufs) & 1) ^ 1, p.status)) { ok = false; break; }
          for (int c = 0; c < nkc; ++c) {
            if (!mbar_wait(&bars->k_full[ksl], kph, p.status)) { ok = false; break; }
            tc_fence_after_sync();
            const uint64_t kd = kd0 + ksl * (slot_bytes >> 4);
            const uint64_t qd = p.q_stream ? kd + (kChunkBytes >> 4) : qd0 + c * (kChunkBytes >> 4);
            umma_bf16_ss(d, qd, kd, idesc_qk, c != 0);
            if (c + 1 < nkc || tail == 4) {
              umma_bf16_ss(d, qd + 2, kd + 2, idesc_qk, 1);
              umma_bf16_ss(d, qd + 4, kd + 4, idesc_qk, 1);
              umma_bf16_ss(d, qd + 6, kd + 6, idesc_qk, 1);
            } else {
              for (int kk = 1; kk < tail; ++kk) umma_bf16_ss(d, qd + 2 * kk, kd + 2 * kk, idesc_qk, 1);
            }
            umma_commit(&bars->k_empty[ksl]);
            if (++ksl == p.k_slots) { ksl = 0; kph ^= 1; }
          }
          if (!ok) break;
          umma_commit(&bars->s_full[sb]);
        }
        if (j >= 1) {
          const int i = j - 1, vs = i % p.v_slots, pb = i & 1;
          if (!mbar_wait(&bars->v_full[vs], (i / p.v_slots) & 1, p.status)) { ok = false; break; }
          if (!mbar_wait(&bars->p_full[pb], (i >> 1) & 1, p.status)) { ok = false; break; }
          tc_fence_after_sync();
          const uint64_t vd = vd0 + vs * nvc * (kChunkBytes >> 4);
#pragma unroll
          for (int kk = 0; kk < kBKeys / 16; ++kk)                  // 16 keys: 8 columns of P, 2048 B of V
            umma_bf16_ts(tmem_o, tmem_p + pb * 64 + kk * 8, vd + kk * 128, idesc_pv, (i | kk) != 0);
          umma_commit(&bars->v_empty[vs]);
          umma_commit(&bars->p_empty[pb]);
          if (i == ntiles - 1) umma_commit(&bars->o_full);
        }
      }
    }
  } else {
    const int quarter = warp & 3, half = (warp - 2) >> 2, r = quarter * 32 + lane;
    const uint32_t lane_off = (uint32_t)(quarter * 32) << 16;
    const int q_pos = ctx_off + q0 + r, hi = min(q_pos, seq_len - 1);
    const int lo = first_key(p, q_pos);
    const int warp_pos0 = ctx_off + q0 + quarter * 32;       // position of the warp's first row
    const int warp_lo = first_key(p, warp_pos0 + 31);        // largest lo of its rows
    const int key0 = half * 64;                              // this thread's keys inside a tile
    const float scale2 = p.scale * kLog2e;
    const float* bias = p.bias ? p.bias + (size_t)h * p.bias_len : nullptr;
    const int last = p.bias_len - 1;
    const float far = bias ? bias[last] * kLog2e : 0.f;
    // Window entry e of tile j (from lo_tile) holds the bias of distance d0 - e, d0 = warp_pos0 + 31 - its first key; key k
    // of the tile is entry 31 - lane + k for this row. Tiles that lie wholly beyond the table need none.
    auto tile_near = [&](int j) { return bias && warp_pos0 - ((lo_tile + j) * kBKeys + kBKeys - 1) < last; };
    auto fill_window = [&](int j) {
      const int d0 = warp_pos0 + 31 - (lo_tile + j) * kBKeys;
#pragma unroll
      for (int i = 0; i < 3; ++i) {
        const int e = half * 32 + lane + i * 64;
        if (e < kWin) bars->window[j & 1][quarter][e] = bias[min(max(d0 - e, 0), last)] * kLog2e;
      }
    };
    // m: reference maximum of the row in the log2 domain (the same in both threads of a row), raised
    // lazily, by more than 2^8. The null entry is the state before the first key: score 0, weight 1.
    float m = p.null_entry ? 0.f : -INFINITY, l = (p.null_entry || p.sink) && half == 0 ? 1.f : 0.f;
    if (p.sink) m = p.sink[h] * kLog2e;
    bool ok = true;
    const int vcols = (p.vdim + 31) / 32;
    if (tile_near(0)) fill_window(0);
    pair_sync(quarter);
    for (int j = 0; j < ntiles; ++j) {
      const int sb = j % s_bufs, pb = j & 1, kbase = (lo_tile + j) * kBKeys + key0;
      // after a wait that ran out the warp goes through the motions without waiting, so that its
      // partner is never left at a barrier
      ok = ok && __all_sync(0xffffffffu, mbar_wait(&bars->s_full[sb], (j / s_bufs) & 1, p.status));
      tc_fence_after_sync();
      uint32_t s0[32], s1[32];
      const uint32_t s_addr = tmem_s + sb * kBKeys + key0 + lane_off;
      tmem_ld_32x32b_x32(s_addr, s0);
      tmem_ld_32x32b_x32(s_addr + 32, s1);
      tmem_ld_wait();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->s_empty[sb]);
      if (tile_near(j)) {
        const float* w = bars->window[j & 1][quarter] + 31 - lane + key0;
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          s0[i] = __float_as_uint(fmaf(__uint_as_float(s0[i]), scale2, w[i]));
          s1[i] = __float_as_uint(fmaf(__uint_as_float(s1[i]), scale2, w[i + 32]));
        }
      } else {
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          s0[i] = __float_as_uint(fmaf(__uint_as_float(s0[i]), scale2, far));
          s1[i] = __float_as_uint(fmaf(__uint_as_float(s1[i]), scale2, far));
        }
      }
      if (kbase + 63 > min(warp_pos0, seq_len - 1) || kbase < warp_lo) {                    // (warp-uniform)
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          if (kbase + i > hi || kbase + i < lo) s0[i] = __float_as_uint(-INFINITY);
          if (kbase + 32 + i > hi || kbase + 32 + i < lo) s1[i] = __float_as_uint(-INFINITY);
        }
      }
      float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        mx0 = fmaxf(mx0, __uint_as_float(s0[i]));
        mx1 = fmaxf(mx1, __uint_as_float(s1[i]));
      }
      float tile_max = fmaxf(mx0, mx1);
      bars->row_max[pb][half][r] = tile_max;
      if (j + 1 < ntiles && tile_near(j + 1)) fill_window(j + 1);
      pair_sync(quarter);
      tile_max = fmaxf(tile_max, bars->row_max[pb][half ^ 1][r]);
      float alpha = 1.f;
      bool rescale = false;
      if (tile_max > m + 8.f) {
        if (m != -INFINITY) { alpha = ex2_approx(m - tile_max); rescale = j > 0; }
        m = tile_max;
      }
      const float m_use = m == -INFINITY ? 0.f : m;
      // the P buffer is free once the product of two tiles ago has run
      ok = ok && __all_sync(0xffffffffu, mbar_wait(&bars->p_empty[pb], ((j >> 1) & 1) ^ 1, p.status));
      if (__any_sync(0xffffffffu, rescale)) {
        ok = ok && __all_sync(0xffffffffu, mbar_wait(&bars->p_empty[pb ^ 1], ((j - 1) >> 1) & 1, p.status));
        tc_fence_after_sync();
        for (int c = half; c < vcols; c += 2) {
          uint32_t rr[32];
          tmem_ld_32x32b_x32(tmem_o + lane_off + c * 32, rr);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) rr[i] = __float_as_uint(__uint_as_float(rr[i]) * alpha);
          tmem_st_32x32b_x32(tmem_o + lane_off + c * 32, rr);
        }
      }
      tc_fence_after_sync();
      float rs0 = 0.f, rs1 = 0.f;
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const float a0 = ex2_approx(__uint_as_float(s0[2 * i]) - m_use), a1 = ex2_approx(__uint_as_float(s0[2 * i + 1]) - m_use);
        rs0 += a0;
        rs1 += a1;
        s0[i] = pack_bf16x2(a0, a1);
      }
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const float a0 = ex2_approx(__uint_as_float(s1[2 * i]) - m_use), a1 = ex2_approx(__uint_as_float(s1[2 * i + 1]) - m_use);
        rs0 += a0;
        rs1 += a1;
        s0[16 + i] = pack_bf16x2(a0, a1);
      }
      tmem_st_32x32b_x32(tmem_p + pb * 64 + half * 32 + lane_off, s0);
      tmem_st_wait();
      l = l * alpha + (rs0 + rs1);
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->p_full[pb]);
    }
    bars->row_max[ntiles & 1][half][r] = l;       // (the slot read in the last tile has the other parity)
    pair_sync(quarter);
    l += bars->row_max[ntiles & 1][half ^ 1][r];
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait(&bars->o_full, 0, p.status));
    if (ok) {
      tc_fence_after_sync();
      float inv = l > 0.f ? p.out_scale / l : 0.f;
      if (p.gate && r < rows)
        inv *= sigmoid_f(to_f(reinterpret_cast<const __nv_bfloat16*>(p.gate)[(size_t)(q_begin + q0 + r) * p.ldg + h]));
      __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)(q_begin + q0 + r) * p.ldo + (size_t)h * p.vdim;
      for (int c = half; c < vcols; c += 2) {
        uint32_t rr[32];
        tmem_ld_32x32b_x32(tmem_o + lane_off + c * 32, rr);
        tmem_ld_wait();
        if (r < rows) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (c * 32 + i < p.vdim) {
              uint4 w;
              w.x = pack_bf16x2(__uint_as_float(rr[i + 0]) * inv, __uint_as_float(rr[i + 1]) * inv);
              w.y = pack_bf16x2(__uint_as_float(rr[i + 2]) * inv, __uint_as_float(rr[i + 3]) * inv);
              w.z = pack_bf16x2(__uint_as_float(rr[i + 4]) * inv, __uint_as_float(rr[i + 5]) * inv);
              w.w = pack_bf16x2(__uint_as_float(rr[i + 6]) * inv, __uint_as_float(rr[i + 7]) * inv);
              *reinterpret_cast<uint4*>(dst + c * 32 + i) = w;
            }
          }
        }
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  if (warp == 1) tmem_dealloc(bars->tmem_base, 512);
}

// ------------------------------------------------------------------------------------ host helpers
// Shapes the decode kernel serves. tk: keys per tile; cls: register class (0: 8 output tiles, 2 query
// chunks and 4 heads per warp, 1: 16 tiles, 8 heads, queries in shared memory).
static bool decode_plan(const B200BiasAttn* a, BiasAttnParams& p, size_t& smem, int& tk, int& cls) {
  if (a->grouped || a->chunk || a->window || a->gate || a->scale != 1.f || a->sink || a->out_scale != 1.f) return false;           // (attn_grouped.cu)
  if (a->f32 || (a->kw & 7) || (a->vdim & 7) || (a->ldq & 7) || (a->ldo & 1)) return false;
  if (((uintptr_t)a->q | (uintptr_t)a->cache) & 15) return false;
  const int R = a->H / a->G, nkc = (a->kw + 63) / 64;
  p.mt = (R + 15) / 16;
  // All heads of a request in one CTA read each key once; where they do not fit its registers and shared
  // memory, CTAs share them by kv groups (the keys then come out of L2 for all but the first).
  for (int z = 1; z <= a->G; ++z) {
    if (a->G % z) continue;
    const int G = a->G / z, H = a->H / z, nvc = (G * a->vdim + 63) / 64;
    p.zslices = z;
    p.hp = (H + 15) & ~15;
    const int mtiles = p.hp / 16, heads = p.hp / kDecWarps;         // heads: per warp
    const int per_warp = (G * p.mt * (a->vdim / 8) + kDecWarps - 1) / kDecWarps;
    if (heads > 8 || per_warp > 16) continue;
    // The key row is cut into slices (a power of two, then without empty ones), as many as there are
    // warps for and as the partial sums leave room for.
    int most = 1;
    while (mtiles * most * 2 <= kDecWarps && most * 2 <= nkc) most *= 2;
    for (tk = 32; tk >= 16; tk -= 16) {
      if (a->block_size < 8 || (a->block_size < tk ? tk % a->block_size : a->block_size % tk)) continue;
      for (int slices = most; slices >= 1; slices /= 2) {
        const int cper = (nkc + slices - 1) / slices;
        p.ksplit = (nkc + cper - 1) / cper;
        cls = per_warp <= 8 && cper <= 2 && heads <= 4 ? 0 : 1;
        for (int n = 2 * kDecMaxSlots; n >= 4; --n) {         // slots of both rings together
          p.k_slots = (n + 1) / 2;
          p.v_slots = n / 2;
          smem = (size_t)decode_smem(tk, p.hp, nkc, nvc, G * p.mt * 16, p.ksplit, p.k_slots, p.v_slots, cls == 1).total +
                 1024;
          if (smem <= 227 * 1024) return true;
        }
      }
    }
  }
  return false;
}

static bool prefill_plan(const B200BiasAttn* a, BiasAttnParams& p, size_t& smem) {
  if (a->f32 || !a->tile_req || (a->kw & 7) || (a->vdim & 7) || a->vdim > 256 || (a->ldq & 7) || (a->ldo & 7)) return false;
  if (((uintptr_t)a->q | (uintptr_t)a->cache | (uintptr_t)a->out) & 15 || (a->values_in_keys && !a->grouped)) return false;
  if (((uintptr_t)a->keys | (uintptr_t)a->values | (uintptr_t)a->shared_keys) & 15 || (a->ldk | a->ldv | a->lds) & 7) return false;
  const int bs = a->block_size, maps = a->maps > 1 ? a->maps : 1;
  if (bs < 8 || (bs & 7) || (bs < kBKeys && kBKeys % bs) || (bs > kBKeys && bs % kBKeys)) return false;
  // a group's columns start on a 16-byte boundary and the last product of 16 reads none of the next group
  if (a->grouped && (((a->kw / a->G - a->key_at) / maps & 15) || (a->kw / a->G & 7) || (a->key_at & 7))) return false;
  if (a->shared && (!a->shared_keys || (a->shared & 15) || maps > 1 || !a->grouped)) return false;
  const int nkc = ((a->grouped ? (a->kw / a->G - a->key_at) / maps : a->kw) + 63) / 64 + (a->shared + 63) / 64, nvc = (a->vdim + 63) / 64;
  const int limit = 227 * 1024, fixed = (int)sizeof(BiasPrefillBars) + 1024;
  // the query tile stays in shared memory if enough of the key ring fits beside it
  for (p.q_stream = 0; p.q_stream < 2; ++p.q_stream) {
    const int slot = (p.q_stream ? 2 : 1) * kChunkBytes, resident = p.q_stream ? 0 : nkc * kChunkBytes;
    for (p.v_slots = 2; p.v_slots >= 1; --p.v_slots) {
      const int left = limit - fixed - resident - p.v_slots * nvc * kChunkBytes;
      p.k_slots = left < 0 ? 0 : left / slot;
      if (p.k_slots > kMaxKSlots) p.k_slots = kMaxKSlots;
      if (p.k_slots >= (p.v_slots == 2 ? kMinKSlots + 1 : kMinKSlots)) {
        smem = (size_t)fixed + resident + p.v_slots * nvc * kChunkBytes + p.k_slots * slot;
        return true;
      }
    }
  }
  return false;
}

struct PageMapKey {
  const void* base;
  uint64_t blocks;
  int bs, kw, vw, rows;
  bool operator==(const PageMapKey& o) const {
    return base == o.base && blocks == o.blocks && bs == o.bs && kw == o.kw && vw == o.vw && rows == o.rows;
  }
};
struct PageMapHash {
  size_t operator()(const PageMapKey& k) const {
    return reinterpret_cast<size_t>(k.base) ^ (k.blocks * 0x9e3779b97f4a7c15ull) ^ ((size_t)k.bs << 40) ^
           ((size_t)k.kw << 20) ^ ((size_t)k.vw << 4) ^ (size_t)k.rows;
  }
};

// Tensor maps of the key and the value part of a page, built once per cache; a load brings up to
// `keys` rows of one page.
static bool page_maps(const B200BiasAttn* a, int keys, CUtensorMap* mk, CUtensorMap* mv) {
  static std::mutex mu;
  static std::unordered_map<PageMapKey, std::pair<CUtensorMap, CUtensorMap>, PageMapHash> maps;
  const int vw = a->values_in_keys ? 0 : a->G * a->vdim;
  const uint32_t rows = a->block_size < keys ? a->block_size : keys;
  PageMapKey key{a->cache, (uint64_t)a->num_blocks, a->block_size, a->kw, vw, (int)rows};
  std::lock_guard<std::mutex> lock(mu);
  auto it = maps.find(key);
  if (it == maps.end()) {
    if (maps.size() > 4096) maps.clear();
    const uint64_t page = (uint64_t)a->block_size * (a->kw + vw) * 2;
    const uint8_t* base = reinterpret_cast<const uint8_t*>(a->cache);
    CUtensorMap k, v;
    if (!encode_tmap_3d(&k, base, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a->kw, a->block_size, a->num_blocks,
                        (uint64_t)a->kw * 2, page, 64, rows, 1, CU_TENSOR_MAP_SWIZZLE_128B) ||
        (vw && !encode_tmap_3d(&v, base + (size_t)a->block_size * a->kw * 2, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, vw,
                               a->block_size, a->num_blocks, (uint64_t)vw * 2, page, 64, rows, 1, CU_TENSOR_MAP_SWIZZLE_128B)))
      return false;
    if (!vw) v = k;
    it = maps.emplace(key, std::make_pair(k, v)).first;
  }
  *mk = it->second.first;
  *mv = it->second.second;
  return true;
}

// Tensor maps of key, value and shared rows outside a page tensor.
static bool split_maps(const B200BiasAttn* a, int keys, CUtensorMap* mk, CUtensorMap* mv, CUtensorMap* ms) {
  const uint32_t rows = a->block_size < keys ? a->block_size : keys;
  auto map = [&](CUtensorMap* m, const void* base, long long cols, long long ld) {
    return encode_tmap_3d(m, base, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, cols, a->block_size, a->num_blocks, (uint64_t)ld * 2,
                          (uint64_t)ld * 2 * a->block_size, 64, rows, 1, CU_TENSOR_MAP_SWIZZLE_128B);
  };
  return map(mk, a->keys, a->kw, a->ldk) && map(mv, a->values, (long long)a->G * a->vdim, a->ldv) &&
         (!a->shared || map(ms, a->shared_keys, a->shared, a->lds));
}

static BiasAttnParams common_params(const B200BiasAttn* a) {
  BiasAttnParams p{};
  p.q = a->q; p.ldq = a->ldq; p.out = a->out; p.ldo = a->ldo; p.cache = a->cache;
  p.block_table = (const int32_t*)a->block_table; p.max_blocks = a->max_blocks;
  p.seq_lens = (const int32_t*)a->seq_lens; p.q_start = (const int32_t*)a->q_start;
  p.num_reqs = a->num_reqs; p.rows = a->rows;
  p.H = a->H; p.G = a->G; p.kw = a->kw; p.vdim = a->vdim; p.block_size = a->block_size;
  p.maps = a->maps > 1 ? a->maps : 1; p.window = a->window; p.values_in_keys = a->values_in_keys;
  p.gate = a->gate; p.ldg = a->ldg; p.sink = a->sink; p.out_scale = a->out_scale;
  p.pitch = a->kw / a->G; p.key_at = a->key_at; p.vpitch = a->values_in_keys ? p.pitch : a->vdim;
  p.qw = a->grouped ? (p.pitch - p.key_at) / p.maps : a->kw; p.chunk = a->chunk; p.scale = a->scale;
  p.own_chunks = (p.qw + 63) / 64;
  if (a->shared) p.qw = p.own_chunks * 64 + a->shared;
  p.bias = (const float*)a->bias; p.bias_len = a->bias_len; p.null_entry = a->null_entry;
  p.splits = a->splits < 1 ? 1 : a->splits; p.tmp_o = (float*)a->tmp_o; p.tmp_lse = (float*)a->tmp_lse;
  p.tile_req = (const int32_t*)a->tile_req; p.tile_q0 = (const int32_t*)a->tile_q0;
  p.status = device_status_word();
  return p;
}

template <typename T, int kAnyHeads>
static int launch_any(const BiasAttnParams& p, cudaStream_t stream) {
  if ((long)kAnyHeads * p.vdim > 128l * kAnyAcc) return -4;
  const size_t smem = (size_t)kAnyHeads * (p.qw + kAnyKeys) * 4;
  if (smem > 200 * 1024) return -4;
  static PerDeviceOnce once;
  if (once.first())
    cudaFuncSetAttribute(bias_attn_any_kernel<T, kAnyHeads>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  dim3 grid(p.rows, (p.H + kAnyHeads - 1) / kAnyHeads);
  return launch_pdl(bias_attn_any_kernel<T, kAnyHeads>, grid, dim3(128), smem, stream, p) == cudaSuccess ? 0 : -2;
}
template <typename T>
static int launch_any(const BiasAttnParams& p, cudaStream_t stream) {
  return 4l * p.vdim <= 128l * kAnyAcc && 16l * (p.qw + kAnyKeys) <= 200 * 1024 ? launch_any<T, 4>(p, stream)
                                                                                : launch_any<T, 1>(p, stream);
}

template <int TK, int MAXI, int CPW, int HPW>
static int launch_decode_mma(const B200BiasAttn* a, const BiasAttnParams& p, size_t smem, cudaStream_t stream) {
  CUtensorMap tmK, tmV;
  if (!page_maps(a, TK, &tmK, &tmV)) return -3;
  static PerDeviceOnce once;
  if (once.first())
    cudaFuncSetAttribute(bias_attn_decode_kernel<TK, MAXI, CPW, HPW>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
  return launch_pdl(bias_attn_decode_kernel<TK, MAXI, CPW, HPW>, dim3(p.rows, p.splits, p.zslices), dim3(kDecThreads), smem, stream, tmK, tmV,
                    p) == cudaSuccess ? 0 : -2;
}

template <typename TO, int TOK>
static int launch_mix(const MixParams& p, int gy, cudaStream_t stream) {
  const size_t smem = ((size_t)kMixHeads * p.H + (size_t)TOK * p.H * p.dim) * 4;
  if (smem > 220 * 1024) return -4;
  static PerDeviceOnce once;
  if (once.first())
    cudaFuncSetAttribute(head_mix_kv_kernel<TO, TOK>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  return launch_pdl(head_mix_kv_kernel<TO, TOK>, dim3((p.T + TOK - 1) / TOK, gy), dim3(256), smem, stream, p) ==
                 cudaSuccess ? 0 : -2;
}

template <typename TO, int RR>
static int launch_mix_vec(const MixParams& p, cudaStream_t stream) {
  const int sms = b200_num_sms();
  const long threads = (long)p.T * p.G * p.dim / 4;
  int slices = 1;                          // few tokens: the output heads are dealt out to more blocks
  while (slices < p.H && slices < 16 && (threads + 255) / 256 * slices < 2l * sms) slices *= 2;
  int hpb = (p.H + slices - 1) / slices;
  slices = (p.H + hpb - 1) / hpb;
  const size_t smem = (size_t)hpb * p.H * 4;
  if (smem > 96 * 1024) return -5;         // (the caller takes the other kernel)
  static PerDeviceOnce once;
  if (once.first())
    cudaFuncSetAttribute(head_mix_kv_vec_kernel<TO, RR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024);
  long gx = (threads + 255) / 256;
  if (gx > 16l * sms) gx = 16l * sms;
  return launch_pdl(head_mix_kv_vec_kernel<TO, RR>, dim3((unsigned)gx, slices + 1), dim3(256), smem, stream, p, hpb) ==
                 cudaSuccess ? 0 : -2;
}
template <typename TO>
static int launch_mix_vec(const MixParams& p, cudaStream_t stream) {
  const size_t es = sizeof(TO);
  if ((p.dim & 3) || (p.vdim & 3) || (p.ld & 3) || (p.ldq & 3) || ((uintptr_t)p.qkv & 15) ||
      ((uintptr_t)p.q_out & (4 * es - 1)) || ((uintptr_t)p.cache & (4 * es - 1)))
    return -5;
  switch (p.H / p.G) {
    case 1: return launch_mix_vec<TO, 1>(p, stream);
    case 2: return launch_mix_vec<TO, 2>(p, stream);
    case 3: return launch_mix_vec<TO, 3>(p, stream);
    case 4: return launch_mix_vec<TO, 4>(p, stream);
    case 6: return launch_mix_vec<TO, 6>(p, stream);
    case 8: return launch_mix_vec<TO, 8>(p, stream);
    case 12: return launch_mix_vec<TO, 12>(p, stream);
    case 16: return launch_mix_vec<TO, 16>(p, stream);
    default: return -5;
  }
}

static bool valid_args(const B200BiasAttn* a) {
  return a->H > 0 && a->G > 0 && a->H % a->G == 0 && a->kw > 0 && a->vdim > 0 && a->block_size > 0 &&
         (!a->bias || a->bias_len > 0) && (!a->grouped || a->kw % a->G == 0) && a->chunk >= 0 &&
         a->window >= 0 && (a->maps <= 1 || (a->grouped && a->kw / a->G % a->maps == 0 && a->H / a->G % a->maps == 0)) &&
         (!a->values_in_keys || a->vdim <= a->kw / a->G) && !(a->sink && a->null_entry) &&
         (!a->key_at || (a->values_in_keys && a->grouped && a->maps <= 1 && a->key_at > 0 && a->key_at < a->kw / a->G));
}

}  // namespace b200

using namespace b200;

extern "C" {

int b200_head_mix_kv(const void* qkv, long long ld, const void* mix, void* q_out, long long ldq, const void* slots,
                     void* cache, int H, int G, int dim, int vdim, int block_size, int T, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dim <= 0 || vdim <= 0 || block_size <= 0) return -1;
  MixParams p{(const float*)qkv, ld, (const float*)mix, q_out, ldq, (const int64_t*)slots, cache, H, G, dim, vdim,
              block_size, T};
  const int rc = f32 ? launch_mix_vec<float>(p, stream) : launch_mix_vec<__nv_bfloat16>(p, stream);
  if (rc != -5) return rc;
  // few tokens: one per CTA, so that more SMs take part
  const int gy = (H + kMixHeads - 1) / kMixHeads;
  const size_t wide = ((size_t)kMixHeads * H + 4 * (size_t)H * dim) * 4;
  const bool narrow = wide > 220 * 1024 || (long)((T + 3) / 4) * gy < 2l * b200_num_sms();
  if (f32) return narrow ? launch_mix<float, 1>(p, gy, stream) : launch_mix<float, 4>(p, gy, stream);
  return narrow ? launch_mix<__nv_bfloat16, 1>(p, gy, stream) : launch_mix<__nv_bfloat16, 4>(p, gy, stream);
}

// 2: tensor-core kernels for this shape, 1: the any-size kernel only. phase 0 decode, 1 prefill.
int b200_bias_attn_kernel(const B200BiasAttn* a, int phase) {
  BiasAttnParams p{};
  size_t smem;
  int tk, cls;
  if (!valid_args(a)) return 0;
  if (phase == 0) return decode_plan(a, p, smem, tk, cls) || grouped_decode_fits(a) ? 2 : 1;
  return prefill_plan(a, p, smem) ? 2 : 1;
}

int b200_bias_attn_decode(const B200BiasAttn* a, int any_size, cudaStream_t stream) {
  if (a->rows <= 0) return 0;
  if (!valid_args(a)) return -1;
  BiasAttnParams p = common_params(a);
  p.q_start = nullptr;
  size_t smem;
  int tk, cls;
  if (!any_size && grouped_decode_fits(a)) return grouped_decode(a, stream);
  if (any_size || !decode_plan(a, p, smem, tk, cls))
    return a->f32 ? launch_any<float>(p, stream) : launch_any<__nv_bfloat16>(p, stream);
  if (p.splits > 1 && (!p.tmp_o || !p.tmp_lse)) return -1;
  const int rc = tk == 32 ? (cls == 0 ? launch_decode_mma<32, 8, 2, 4>(a, p, smem, stream)
                                      : launch_decode_mma<32, 16, 0, 8>(a, p, smem, stream))
                          : (cls == 0 ? launch_decode_mma<16, 8, 2, 4>(a, p, smem, stream)
                                      : launch_decode_mma<16, 16, 0, 8>(a, p, smem, stream));
  if (rc || p.splits == 1) return rc;
  return b200_attn_decode_merge(p.tmp_o, p.tmp_lse, p.out, (int)p.ldo, p.rows, p.H, p.vdim, p.splits, stream);
}

int b200_bias_attn_prefill(const B200BiasAttn* a, int any_size, cudaStream_t stream) {
  if (a->rows <= 0) return 0;
  if (!valid_args(a) || !a->q_start) return -1;
  BiasAttnParams p = common_params(a);
  size_t smem;
  const bool split = a->keys != nullptr;
  if (any_size || !prefill_plan(a, p, smem)) {
    if (split || a->shared) return -4;
    return a->f32 ? launch_any<float>(p, stream) : launch_any<__nv_bfloat16>(p, stream);
  }
  if (a->num_tiles <= 0) return 0;
  CUtensorMap tmQ, tmK, tmV, tmS;
  if (!encode_tmap_2d(&tmQ, a->q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (uint64_t)a->rows, (uint64_t)a->H * p.qw,
                      (uint64_t)a->ldq, kBQ, 64, CU_TENSOR_MAP_SWIZZLE_128B) ||
      !(split ? split_maps(a, kBKeys, &tmK, &tmV, &tmS) : page_maps(a, kBKeys, &tmK, &tmV)))
    return -3;
  if (!a->shared) tmS = tmK;
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(bias_attn_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
  bias_attn_prefill_kernel<<<dim3(a->num_tiles, a->H), kPrefillThreads, smem, stream>>>(tmQ, tmK, tmV, tmS, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // extern "C"
