// Prompt portions of the recurrences over outer products (outer.cu) in chunks of 64 tokens, D <= 256, at fp32 accuracy
// on the tensor cores: fp32 operands are kept as bf16 pairs (x = hi + lo, products hi hi + hi lo + lo hi); operands
// that arrive as bf16 are used as they are.
//
// With G_i the sum of the log decays up to token i inside a chunk (per key channel, or one per head) and S the state
// before it,
//   o_i = (q_i e^(G_i))^T S + sum_{j <= i} P_ij v_j,   P_ij = sum_d q_id k_jd e^(G_id - G_jd)
//   S <- e^(G_last) S + sum_j (k_j e^(G_last - G_j)) v_j^T
// (the chunkwise forms; Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training"; Dao and Gu,
// "Transformers are SSMs").
//
//   outer_pairs_channel_kernel, outer_pairs_head_kernel   what does not depend on the state, parallel over chunks.
//       Decay per channel (kind 0): q' = q e^G, k' = k e^(G_last - G) and P as pairs, G_last. P is the product of q' and
//       k e^-G while no channel fades by more than 2^-86 inside the chunk, else summed term by term. Decay per head
//       (kind 1): P = q k^T times e^(G_i - G_j) dt_j as pairs, e^G and dt e^(G_last - G); q k^T once for the heads that
//       share it
//   outer_scan_kernel   per (64 value columns, head, segment of a portion): walks the chunks with S in registers, as the
//       accumulators of its update; two block barriers a chunk, the next chunk's operands under way by cp.async
//
// A portion may be cut into segments of ``seg_tiles`` 128-row tiles, whose CTAs run side by side in two launches of the scan.
// The first runs segment 0 and leaves the state behind it, and for the segments in between the state they would leave if
// they started from zero, with their decay. The second runs the segments from 1 on, each from the state that it puts
// together from those. Only the last one writes the slot's state, which nobody reads any more.
//
// Rows past the end of a portion are zeros with decay one. P is lower triangular: of row block b (16 rows) only the first
// 16 (b + 1) columns exist.
#include "api.h"
#include "sm100.cuh"

namespace b200 {

typedef __nv_bfloat16 bf16;
bool outer_ok(const B200Outer* a);

static constexpr int kC = 64;                    // tokens per chunk
static constexpr int kVs = 64;                   // value columns per CTA of the scan
static constexpr int kPairThreads = 256, kScanThreads = 512;
static constexpr int kPlane = kC * 128;          // bytes of a 64 x 64 bf16 plane
static constexpr float kLog2e = 1.4426950408889634f;
// kind 0, in powers of two: of a chunk whose factors are taken apart; of one token (beyond, nothing of the state is left)
static constexpr float kMostDecay = 86.f, kTokenDecay = 44.f;
static constexpr int kHeadsPerPair = 8;          // heads that one CTA of the head pairs serves

__device__ __forceinline__ void oc_ldsm4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void oc_ldsm4t(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void oc_mma(float* d, const uint32_t* a, const uint32_t* b) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
// d += a b for N 8-column tiles
template <int N>
__device__ __forceinline__ void oc_mman(float (*d)[4], const uint32_t* a, const uint32_t* b) {
#pragma unroll
  for (int n = 0; n < N; ++n) oc_mma(d[n], a, b + 2 * n);
}
__device__ __forceinline__ void oc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(x - h.x, y - h.y);
}
__device__ __forceinline__ void oc_cp16(uint32_t dst, const void* src, bool real) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(real ? 16 : 0) : "memory");
}
__device__ __forceinline__ void oc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void oc_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ float oc_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float oc_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// byte offset of 16-byte unit ``u`` of row ``r`` in a plane of 128-byte rows (units xored by the row)
__device__ __forceinline__ uint32_t oc_unit(int r, int u) { return (uint32_t)(r * 128 + ((u ^ (r & 7)) << 4)); }
// the address a lane gives ldmatrix.trans for a 16 (k) x 16 (n) block of such a plane at (k0, n0)
__device__ __forceinline__ uint32_t oc_b(uint32_t base, int k0, int n0, int lane) {
  return base + oc_unit(k0 + (lane & 15), (n0 >> 3) + (lane >> 4));
}

// Workspace of one chunk and head, in bf16 values: kind 0: q' hi | lo | k' hi | lo ([64][D] each) | P hi | lo ([64][64]),
// kind 1: P hi | lo. Factors in fp32: kind 0: G_last (to base 2) [D], kind 1: e^G [64] | dt e^(G_last - G) [64].
__host__ __device__ inline size_t pair_values(int kind, int D) { return (kind == 0 ? (size_t)4 * kC * D : 0) + 2 * kC * kC; }
__host__ __device__ inline int factor_values(int kind, int D) { return kind == 0 ? D : 2 * kC; }

// Chunks of the portions ahead of ``req`` (all lanes of a warp).
__device__ __forceinline__ int chunks_ahead(const B200Rows& R, int req, int lane) {
  int n = 0;
  for (int i = lane; i < req; i += 32) n += (R.q_start[i + 1] - R.q_start[i] + kC - 1) / kC;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) n += __shfl_xor_sync(0xffffffffu, n, o);
  return n;
}

// ------------------------------------------------------------------------------------- pairs, decay per channel
struct ChannelSmem { int q, k, a1, e, total; };
__host__ __device__ inline ChannelSmem channel_smem(int D, int rank) {
  ChannelSmem m;
  const int rows = kC * (D + 8) * 2;             // a plane of q' or k e^-G rows
  m.q = 0;
  m.k = 2 * rows;                                // (over both, where P is summed term by term: fp32 [64][D] and [4][D])
  m.a1 = 4 * rows;
  m.e = m.a1 + kC * (rank + 8) * 2;              // 2^(G_last) [D]
  m.total = m.e + D * 4;
  return m;
}

// grid (H, 2 per 128-row tile). Warp w: 16-channel strips w, w + 8, ... of q' and k', half by half; rows 16 (w % 4), columns 32 (w / 4) of P.
__global__ void __launch_bounds__(kPairThreads, 3) outer_pairs_channel_kernel(B200Outer p) {
  extern __shared__ uint8_t pairs_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(pairs_raw) + 127) & ~uintptr_t(127));
  const int D = p.D, rank = p.rank, stride = (D + 8) * 2, plane = kC * stride, astride = (rank + 8) * 2;
  const ChannelSmem L = channel_smem(D, rank);
  const uint32_t base = smem_u32(smem);
  pdl_wait();
  pdl_launch_dependents();
  const B200Rows& R = p.rows;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x, tile = blockIdx.y >> 1;
  const int req = R.tile_req[tile], q0 = R.tile_q0[tile] + (blockIdx.y & 1) * kC, begin = R.q_start[req];
  const int n = min(kC, R.q_start[req + 1] - begin - q0), t0 = R.nd + begin + q0;
  if (n <= 0 || R.slots[R.nd + req] < 0) return;
  const size_t at = (size_t)(chunks_ahead(R, req, lane) + q0 / kC) * p.H + h;
  bf16* wq = reinterpret_cast<bf16*>(p.pairs) + at * pair_values(0, D);
  bf16* wk = wq + 2 * kC * D;
  bf16* wp = wk + 2 * kC * D;
  const bf16* gq = reinterpret_cast<const bf16*>(p.q) + (size_t)t0 * p.ld + (size_t)h * D;      // (kind 0: a key head per state)
  const bf16* gk = reinterpret_cast<const bf16*>(p.k) + (size_t)t0 * p.ld + (size_t)h * D;
  {
    const int units = rank / 8;
    const bf16* a1 = reinterpret_cast<const bf16*>(p.a1);
    for (int x = tid; x < kC * units; x += kPairThreads) {
      const int r = x / units, u = x - r * units;
      oc_cp16(base + L.a1 + r * astride + u * 16, a1 + (size_t)(t0 + (r < n ? r : 0)) * p.lda1 + u * 8, r < n);
    }
    oc_commit();
    oc_wait<0>();
    __syncthreads();
  }
  const int col = (lane & 3) * 2, row = lane >> 2;
  float* sg = reinterpret_cast<float*>(smem);                     // term by term: sums inside blocks of 16 rows [64][D],
  float* st = sg + kC * D;                                       // sums of the blocks [4][D]
  float* se = reinterpret_cast<float*>(smem + L.e);
  // Log decays (to base 2), summed inside blocks of 16 rows; q' and k e^-G (``terms``: those sums, and k' to the workspace).
  const float scale = p.inv_tau * kLog2e;
  auto strips = [&](bool terms) {
    int far = 0;
    for (int u = warp * 2; u < D / 8; u += u & 1 ? 2 * (kPairThreads / 32) - 1 : 1) {    // (neighbours one after the other)
      const int cb = u * 8 + col;                // channels cb, cb + 1
      uint32_t qv[4][2], kv[4][2];
#pragma unroll
      for (int mb = 0; mb < 4; ++mb)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = mb * 16 + half * 8 + row;
          kv[mb][half] = r < n ? *reinterpret_cast<const uint32_t*>(gk + (size_t)r * p.ld + cb) : 0u;
          qv[mb][half] = r < n ? *reinterpret_cast<const uint32_t*>(gq + (size_t)r * p.ld + cb) : 0u;
        }
      float z[4][4];
      const float2 bias = *reinterpret_cast<const float2*>(p.a2b + (size_t)h * D + cb);
#pragma unroll
      for (int mb = 0; mb < 4; ++mb) { z[mb][0] = z[mb][2] = bias.x; z[mb][1] = z[mb][3] = bias.y; }
      const bf16* a2 = reinterpret_cast<const bf16*>(p.a2) + ((size_t)h * D + u * 8 + row) * rank + col;
      for (int k0 = 0; k0 < rank; k0 += 16) {
        const uint32_t w[2] = {*reinterpret_cast<const uint32_t*>(a2 + k0), *reinterpret_cast<const uint32_t*>(a2 + k0 + 8)};
#pragma unroll
        for (int mb = 0; mb < 4; ++mb) {
          uint32_t a[4];
          oc_ldsm4(a, base + L.a1 + (mb * 16 + (lane & 15)) * astride + (lane >> 4) * 16 + k0 * 2);
          oc_mma(z[mb], a, w);
        }
      }
      float block[4][2];                         // sums of the blocks (eight lanes, four apart, hold consecutive rows)
#pragma unroll
      for (int mb = 0; mb < 4; ++mb)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float carry = 0.f;
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            float x = z[mb][half * 2 + e];
            x = mb * 16 + half * 8 + row < n ? fmaxf(-(fmaxf(-x, 0.f) + log1pf(__expf(-fabsf(x)))) * scale, -kTokenDecay) : 0.f;
#pragma unroll
            for (int o = 4; o < 32; o <<= 1) {
              const float y = __shfl_up_sync(0xffffffffu, x, o);
              if (lane >= o) x += y;
            }
            x += carry;
            carry = __shfl_sync(0xffffffffu, x, 28 + (lane & 3));
            z[mb][half * 2 + e] = x;
          }
          block[mb][e] = carry;
        }
      if (terms) {
#pragma unroll
        for (int mb = 0; mb < 4; ++mb) {
          float after[2] = {0.f, 0.f};           // (sums of the blocks behind, not a difference of sums)
#pragma unroll
          for (int x = mb + 1; x < 4; ++x) { after[0] += block[x][0]; after[1] += block[x][1]; }
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int r = mb * 16 + half * 8 + row;
            const float g0 = z[mb][half * 2], g1 = z[mb][half * 2 + 1];
            const float2 kk = unpack_bf16x2(kv[mb][half]);
            *reinterpret_cast<float2*>(sg + r * D + cb) = make_float2(g0, g1);
            uint32_t hi, lo;
            oc_split(kk.x * oc_ex2(block[mb][0] - g0 + after[0]), kk.y * oc_ex2(block[mb][1] - g1 + after[1]), hi, lo);
            *reinterpret_cast<uint32_t*>(wk + (size_t)r * D + cb) = hi;
            *reinterpret_cast<uint32_t*>(wk + kC * D + (size_t)r * D + cb) = lo;
          }
          if (lane < 4) *reinterpret_cast<float2*>(st + mb * D + cb) = make_float2(block[mb][0], block[mb][1]);
        }
        continue;
      }
      float before[2] = {0.f, 0.f};
      const float all0 = block[0][0] + block[1][0] + block[2][0] + block[3][0], all1 = block[0][1] + block[1][1] + block[2][1] + block[3][1];
      if (all0 < -kMostDecay || all1 < -kMostDecay) far = 1;
      if (lane < 4) {
        *reinterpret_cast<float2*>(p.factors + at * D + cb) = make_float2(all0, all1);
        *reinterpret_cast<float2*>(se + cb) = make_float2(oc_ex2(all0), oc_ex2(all1));
      }
#pragma unroll
      for (int mb = 0; mb < 4; ++mb) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const float s0 = before[0] + z[mb][half * 2], s1 = before[1] + z[mb][half * 2 + 1];
          const float2 kk = unpack_bf16x2(kv[mb][half]), qq = unpack_bf16x2(qv[mb][half]);
          uint32_t hi, lo;
          uint8_t* dst = smem + (mb * 16 + half * 8 + row) * stride + cb * 2;
          oc_split(kk.x * oc_ex2(-s0), kk.y * oc_ex2(-s1), hi, lo);
          *reinterpret_cast<uint32_t*>(dst + L.k) = hi;
          *reinterpret_cast<uint32_t*>(dst + L.k + plane) = lo;
          oc_split(p.q_scale * qq.x * oc_ex2(s0), p.q_scale * qq.y * oc_ex2(s1), hi, lo);
          *reinterpret_cast<uint32_t*>(dst + L.q) = hi;
          *reinterpret_cast<uint32_t*>(dst + L.q + plane) = lo;
        }
        before[0] += block[mb][0];
        before[1] += block[mb][1];
      }
    }
    return far;
  };
  const bool far = __syncthreads_or(strips(false));
  // To the workspace in whole rows: q', and k' as k e^-G times e^(G_last).
  for (int x = tid; x < kC * (D / 8); x += kPairThreads) {
    const int r = x / (D / 8), u = x - r * (D / 8);
    const uint8_t* from = smem + r * stride + u * 16;
    const size_t to = (size_t)r * D + u * 8;
    *reinterpret_cast<uint4*>(wq + to) = *reinterpret_cast<const uint4*>(from + L.q);
    *reinterpret_cast<uint4*>(wq + kC * D + to) = *reinterpret_cast<const uint4*>(from + L.q + plane);
    if (far) continue;
    const uint4 a = *reinterpret_cast<const uint4*>(from + L.k), b = *reinterpret_cast<const uint4*>(from + L.k + plane);
    const float4 e0 = *reinterpret_cast<const float4*>(se + u * 8), e1 = *reinterpret_cast<const float4*>(se + u * 8 + 4);
    const float e[8] = {e0.x, e0.y, e0.z, e0.w, e1.x, e1.y, e1.z, e1.w};
    const uint32_t h[4] = {a.x, a.y, a.z, a.w}, l[4] = {b.x, b.y, b.z, b.w};
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 y = unpack_bf16x2(h[i]), z = unpack_bf16x2(l[i]);
      oc_split((y.x + z.x) * e[2 * i], (y.y + z.y) * e[2 * i + 1], hi[i], lo[i]);
    }
    *reinterpret_cast<uint4*>(wk + to) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(wk + kC * D + to) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  if (!far) {
    const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 32;
    if (n0 > m0) return;                         // (blocks above the diagonal are not needed)
    float px[4][4];
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) px[x][e] = 0.f;
    const uint32_t arow = base + L.q + (m0 + (lane & 15)) * stride + (lane >> 4) * 16;
    // B = K^T: the k index runs along K's rows, so no transpose: lanes give rows n, halves k
    const uint32_t brow = base + L.k + (n0 + (lane & 7) + ((lane >> 4) << 3)) * stride + ((lane >> 3) & 1) * 16;
    for (int k0 = 0; k0 < D; k0 += 16) {
      uint32_t qh[4], ql[4], bh[8], bl[8];
      oc_ldsm4(qh, arow + k0 * 2);
      oc_ldsm4(ql, arow + plane + k0 * 2);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        oc_ldsm4(bh + 4 * x, brow + x * 16 * stride + k0 * 2);
        oc_ldsm4(bl + 4 * x, brow + plane + x * 16 * stride + k0 * 2);
      }
      oc_mman<4>(px, qh, bh);
      oc_mman<4>(px, qh, bl);
      oc_mman<4>(px, ql, bh);
    }
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int j = n0 + x * 8 + col;
      if (j >= m0 + 16) continue;                // (beyond the row block's columns)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = m0 + row + half * 8;
        uint32_t hi, lo;
        oc_split(j <= i ? px[x][half * 2] : 0.f, j + 1 <= i ? px[x][half * 2 + 1] : 0.f, hi, lo);
        *reinterpret_cast<uint32_t*>(wp + i * kC + j) = hi;
        *reinterpret_cast<uint32_t*>(wp + kC * kC + i * kC + j) = lo;
      }
    }
    return;
  }
  // Term by term: four threads a row.
  __syncthreads();
  strips(true);
  __syncthreads();
  const int i = tid >> 2, bi = i >> 4;
  for (int j = tid & 3; j < (bi + 1) * 16; j += 4) {
    const int bj = j >> 4;
    float s = 0.f;
    if (j <= i && i < n)
      for (int d = 0; d < D; ++d) {
        float g = sg[i * D + d];
        if (bi == bj) {
          g -= sg[j * D + d];
        } else {
          g += st[bj * D + d] - sg[j * D + d];
          for (int b = bj + 1; b < bi; ++b) g += st[b * D + d];
        }
        s = fmaf(__bfloat162float(gq[(size_t)i * p.ld + d]) * __bfloat162float(gk[(size_t)j * p.ld + d]), oc_ex2(g), s);
      }
    s *= p.q_scale;
    const bf16 hi = __float2bfloat16(s);
    wp[i * kC + j] = hi;
    wp[kC * kC + i * kC + j] = __float2bfloat16(s - __bfloat162float(hi));
  }
}

// ---------------------------------------------------------------------------------------- pairs, decay per head
// grid (G, 2 per 128-row tile, slices of the heads that share a key). Warp w sums up the decays of head w; rows 16 (w % 4),
// columns 32 (w / 4) of every head's P.
__global__ void __launch_bounds__(kPairThreads) outer_pairs_head_kernel(B200Outer p) {
  extern __shared__ uint8_t heads_raw[];
  __shared__ float s_g[kHeadsPerPair][kC], s_dt[kHeadsPerPair][kC];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(heads_raw) + 127) & ~uintptr_t(127));
  const int D = p.D, stride = (D + 8) * 2, plane = kC * stride, share = p.H / p.G;
  const uint32_t sq = smem_u32(smem), sk = sq + plane;
  pdl_wait();
  pdl_launch_dependents();
  const B200Rows& R = p.rows;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = blockIdx.x, tile = blockIdx.y >> 1;
  const int req = R.tile_req[tile], q0 = R.tile_q0[tile] + (blockIdx.y & 1) * kC, begin = R.q_start[req];
  const int n = min(kC, R.q_start[req + 1] - begin - q0), t0 = R.nd + begin + q0;
  if (n <= 0 || R.slots[R.nd + req] < 0) return;
  const int h0 = g * share + blockIdx.z * kHeadsPerPair, nh = min(kHeadsPerPair, share - (int)blockIdx.z * kHeadsPerPair);
  const size_t at = (size_t)(chunks_ahead(R, req, lane) + q0 / kC) * p.H + h0;
  {
    const int units = D / 8;
    const bf16* gq = reinterpret_cast<const bf16*>(p.q) + (size_t)g * D;
    const bf16* gk = reinterpret_cast<const bf16*>(p.k) + (size_t)g * D;
    for (int x = tid; x < kC * units; x += kPairThreads) {
      const int r = x / units, u = x - r * units;
      const size_t from = (size_t)(t0 + (r < n ? r : 0)) * p.ld + u * 8;
      oc_cp16(sq + r * stride + u * 16, gq + from, r < n);
      oc_cp16(sk + r * stride + u * 16, gk + from, r < n);
    }
    oc_commit();
  }
  if (warp < nh) {
    const int h = h0 + warp;
    const float a = p.A[h], bias = p.dt_bias[h];
    float carry = 0.f, gs[2], dts[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int i = x * 32 + lane;
      float dt = 0.f;
      if (i < n) dt = oc_softplus(__bfloat162float(reinterpret_cast<const bf16*>(p.dt)[(size_t)(t0 + i) * p.lddt + h]) + bias);
      float s = -a * dt;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += y;
      }
      s += carry;
      carry = __shfl_sync(0xffffffffu, s, 31);
      gs[x] = s;
      dts[x] = dt;
      s_g[warp][i] = s;
      s_dt[warp][i] = dt;
    }
    float* f = p.factors + (at + warp) * 2 * kC;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      f[x * 32 + lane] = expf(gs[x]);
      f[kC + x * 32 + lane] = dts[x] * expf(carry - gs[x]);
    }
  }
  oc_wait<0>();
  __syncthreads();
  const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 32, col = (lane & 3) * 2, row = lane >> 2;
  if (n0 > m0) return;                           // (blocks above the diagonal are not needed)
  float px[4][4];
#pragma unroll
  for (int x = 0; x < 4; ++x)
#pragma unroll
    for (int e = 0; e < 4; ++e) px[x][e] = 0.f;
  const uint32_t arow = sq + (m0 + (lane & 15)) * stride + (lane >> 4) * 16;
  const uint32_t brow = sk + (n0 + (lane & 7) + ((lane >> 4) << 3)) * stride + ((lane >> 3) & 1) * 16;
  for (int k0 = 0; k0 < D; k0 += 16) {
    uint32_t a[4], b[8];
    oc_ldsm4(a, arow + k0 * 2);
    oc_ldsm4(b, brow + k0 * 2);
    oc_ldsm4(b + 4, brow + 16 * stride + k0 * 2);
    oc_mman<4>(px, a, b);
  }
  for (int h = 0; h < nh; ++h) {
    bf16* wp = reinterpret_cast<bf16*>(p.pairs) + (at + h) * pair_values(1, D);
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int j = n0 + x * 8 + col;
      if (j >= m0 + 16) continue;                // (beyond the row block's columns)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = m0 + row + half * 8;
        const float gi = s_g[h][i];
        const float y0 = j <= i ? px[x][half * 2] * expf(gi - s_g[h][j]) * s_dt[h][j] : 0.f;
        const float y1 = j + 1 <= i ? px[x][half * 2 + 1] * expf(gi - s_g[h][j + 1]) * s_dt[h][j + 1] : 0.f;
        uint32_t hi, lo;
        oc_split(y0, y1, hi, lo);
        *reinterpret_cast<uint32_t*>(wp + i * kC + j) = hi;
        *reinterpret_cast<uint32_t*>(wp + kC * kC + i * kC + j) = lo;
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------------- scan
struct ScanSmem { int s, w, q, k, p, v, f, buf, bufs, total; };     // q .. f: offsets in a buffer
__host__ __device__ inline ScanSmem scan_smem(int kind, int D) {
  ScanSmem m;
  const int rows = kC * (D + 8) * 2, planes = kind == 0 ? 2 : 1;
  int o = 0;
  m.q = o; o += planes * rows;
  m.k = o; o += planes * rows;
  m.p = o; o += 2 * kPlane;
  m.v = o; o += kPlane;
  m.f = o; o += factor_values(kind, D) * 4;
  m.buf = o;
  m.s = 0;
  m.w = 2 * D * 128;
  const int fixed = m.w + (kind == 1 ? 2 * kPlane : 0);
  m.bufs = fixed + 2 * m.buf + 128 <= 227 * 1024 ? 2 : 1;
  m.total = fixed + m.bufs * m.buf;
  return m;
}

// grid (64-wide slices of V, H, 128-row tiles; those where no segment starts return). Warp w: rows 16 (w % 4), columns
// 16 (w / 4) of the 64 x 64 outputs; of the state, 16 x 32 pieces w, w + 16, ... (row block piece / 2, column half
// piece % 2), MI of them at most.
template <int KIND, int MI>
__global__ void __launch_bounds__(kScanThreads, 1) outer_scan_kernel(B200Outer p, int phase) {
  extern __shared__ uint8_t scan_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(scan_raw) + 127) & ~uintptr_t(127));
  const int D = p.D, V = p.V, stride = (D + 8) * 2, plane = kC * stride, splane = D * 128;
  const ScanSmem L = scan_smem(KIND, D);
  const uint32_t base = smem_u32(smem), bufs = base + L.w + (KIND == 1 ? 2 * kPlane : 0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int v0 = blockIdx.x * kVs, h = blockIdx.y, g = h / (p.H / p.G);
  pdl_wait();
  pdl_launch_dependents();
  const B200Rows& R = p.rows;
  const int tile = blockIdx.z, req = R.tile_req[tile], q0 = R.tile_q0[tile];
  if ((q0 / 128) % p.seg_tiles) return;
  const int begin = R.q_start[req], len = R.q_start[req + 1] - begin, span = 128 * p.seg_tiles;
  const int slot = R.slots[R.nd + req], seg = q0 / span, segs = (len + span - 1) / span;
  const bool last = seg == segs - 1, whole = phase == 0 ? seg == 0 : seg > 0;        // whole: with outputs
  if (slot < 0 || len <= 0 || (phase == 0 ? seg > 0 && last : seg == 0)) return;
  int ws0 = 0;                                   // segments of the cut portions ahead
  if (segs > 1) {
    for (int i = lane; i < req; i += 32) {
      const int n = (R.q_start[i + 1] - R.q_start[i] + span - 1) / span;
      ws0 += n > 1 ? n : 0;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ws0 += __shfl_xor_sync(0xffffffffu, ws0, o);
  }
  const int rows = min(len - q0, span), chunks = (rows + kC - 1) / kC, t_base = R.nd + begin + q0;
  const size_t chunk0 = (size_t)chunks_ahead(R, req, lane) + q0 / kC;
  const bool init = R.seq_lens[R.nd + req] > len;
  const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 16, col = (lane & 3) * 2;
  const bf16* gq = reinterpret_cast<const bf16*>(p.q) + (size_t)g * D;
  const bf16* gk = reinterpret_cast<const bf16*>(p.k) + (size_t)g * D;
  const bf16* gv = reinterpret_cast<const bf16*>(p.v) + (size_t)h * V + v0;
  auto fetch = [&](int c) {
    if (c < chunks) {
      const int t0 = t_base + c * kC, n = min(kC, rows - c * kC);
      const uint32_t b = bufs + (c % L.bufs) * L.buf;
      const size_t at = (chunk0 + c) * p.H + h;
      const bf16* w = reinterpret_cast<const bf16*>(p.pairs) + at * pair_values(KIND, D);
      const float* f = p.factors + at * factor_values(KIND, D);
      for (int x = tid; x < kC * 8; x += kScanThreads) {
        const int r = x >> 3, u = x & 7;
        const bool real = r < n && v0 + u * 8 < V;
        oc_cp16(b + L.v + oc_unit(r, u), real ? gv + (size_t)(t0 + r) * p.ld + u * 8 : gv, real);
      }
      const int units = D / 8;
      if (KIND == 0) {
        for (int x = tid; x < kC * units; x += kScanThreads) {
          const int r = x / units, u = x - r * units;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const bf16* from = w + (size_t)e * kC * D + (size_t)r * D + u * 8;
            if (whole) oc_cp16(b + L.q + e * plane + r * stride + u * 16, from, true);
            oc_cp16(b + L.k + e * plane + r * stride + u * 16, from + 2 * kC * D, true);
          }
        }
      } else {
        for (int x = tid; x < kC * units; x += kScanThreads) {
          const int r = x / units, u = x - r * units;
          const size_t from = (size_t)(t0 + (r < n ? r : 0)) * p.ld + u * 8;
          if (whole) oc_cp16(b + L.q + r * stride + u * 16, gq + from, r < n);
          oc_cp16(b + L.k + r * stride + u * 16, gk + from, r < n);
        }
      }
      if (whole) {
        const bf16* wp = w + (KIND == 0 ? (size_t)4 * kC * D : 0);
        for (int x = tid; x < 2 * kC * 8; x += kScanThreads) {
          const int e = x >> 9, r = (x >> 3) & 63, u = x & 7;
          if (u < 2 * (r / 16 + 1)) oc_cp16(b + L.p + e * kPlane + oc_unit(r, u), wp + e * kC * kC + r * kC + u * 8, true);
        }
      }
      for (int x = tid; x < factor_values(KIND, D) / 4; x += kScanThreads) oc_cp16(b + L.f + x * 16, f + x * 4, true);
    }
    oc_commit();
  };
  fetch(0);
  const size_t size = (size_t)D * V;
  float* state = p.state + ((size_t)slot * p.H + h) * size + v0;
  float hs[MI][4][4];
  float total[MI][2];                            // log2 of the decay of the rows of this thread's pieces since the segment's start
  auto each_state = [&](auto f) {                // f(value, value, row, column) for pairs of columns
#pragma unroll
    for (int i = 0; i < MI; ++i) {
      const int piece = warp + 16 * i, d0 = (piece >> 1) * 16 + (lane >> 2), c0 = (piece & 1) * 32 + col;
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int d = d0 + half * 8, c = c0 + n * 8;
          if (d < D && v0 + c < V) f(hs[i][n][half * 2], hs[i][n][half * 2 + 1], d, c);
        }
    }
  };
#pragma unroll
  for (int i = 0; i < MI; ++i) {
    total[i][0] = total[i][1] = 0.f;
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) hs[i][n][e] = 0.f;
  }
  if (seg == 0) {
    if (init)
      each_state([&](float& x, float& y, int d, int c) {
        const float2 s = *reinterpret_cast<const float2*>(state + (size_t)d * V + c);
        x = s.x; y = s.y;
      });
  } else if (whole) {
    for (int i = 0; i < seg; ++i) {
      const size_t at = (size_t)(ws0 + i) * p.H + h;
      const float* s = p.ws + at * size + v0;
      const float* w = p.ws_decay + at * D;
      each_state([&](float& x, float& y, int d, int c) {
        const float2 u = *reinterpret_cast<const float2*>(s + (size_t)d * V + c);
        const float f = i == 0 ? 0.f : exp2f(w[d]);
        x = fmaf(f, x, u.x);
        y = fmaf(f, y, u.y);
      });
    }
  }
  auto store_state = [&]() {                     // the state as an operand
#pragma unroll
    for (int i = 0; i < MI; ++i) {
      const int piece = warp + 16 * i, d = (piece >> 1) * 16 + (lane >> 2);
      if (d >= D) continue;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int u = (piece & 1) * 4 + x;
        uint32_t hi, lo;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          oc_split(hs[i][x][half * 2], hs[i][x][half * 2 + 1], hi, lo);
          uint8_t* dst = smem + L.s + oc_unit(d + half * 8, u) + col * 2;
          *reinterpret_cast<uint32_t*>(dst) = hi;
          *reinterpret_cast<uint32_t*>(dst + splane) = lo;
        }
      }
    }
  };
  if (whole) store_state();
  oc_wait<0>();
  __syncthreads();

  const uint32_t arow = (m0 + (lane & 15)) * stride + (lane >> 4) * 16;
  const uint32_t krow = ((lane & 7) + (lane >> 4) * 8) * stride + ((lane >> 3) & 1) * 16;
  const int i0 = m0 + (lane >> 2), i1 = i0 + 8;
  for (int c = 0; c < chunks; ++c) {
    const int t0 = t_base + c * kC, n = min(kC, rows - c * kC);
    const uint32_t b = bufs + (c % L.bufs) * L.buf, sq = b + L.q, sk = b + L.k, sv = b + L.v;
    const float* f = reinterpret_cast<const float*>(smem + (b - base) + L.f);
    if (L.bufs == 2) fetch(c + 1);
    if (KIND == 1) {                             // v rows with their weights, as pairs
      for (int x = tid; x < kC * 32; x += kScanThreads) {
        const int r = x >> 5, cc = (x & 31) * 2;
        const uint32_t off = oc_unit(r, cc >> 3) + (cc & 7) * 2;
        const float2 y = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(smem + (sv - base) + off));
        const float w = f[kC + r];
        uint32_t hi, lo;
        oc_split(w * y.x, w * y.y, hi, lo);
        *reinterpret_cast<uint32_t*>(smem + L.w + off) = hi;
        *reinterpret_cast<uint32_t*>(smem + L.w + kPlane + off) = lo;
      }
    }
    if (whole) {
      float ox[2][4], ol[2][4];                  // (two sums, to halve the chains of products)
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) ox[x][e] = ol[x][e] = 0.f;
#pragma unroll 4
      for (int k0 = 0; k0 < D; k0 += 16) {
        uint32_t qh[4], ql[4], bh[4], bl[4];
        oc_ldsm4(qh, sq + arow + k0 * 2);
        if (KIND == 0) oc_ldsm4(ql, sq + plane + arow + k0 * 2);
        oc_ldsm4t(bh, oc_b(base + L.s, k0, n0, lane));
        oc_ldsm4t(bl, oc_b(base + L.s + splane, k0, n0, lane));
        oc_mman<2>(ox, qh, bh);
        oc_mman<2>(ol, qh, bl);
        if (KIND == 0) oc_mman<2>(ol, ql, bh);
      }
      const float e0 = KIND == 1 ? f[i0] : 1.f, e1 = KIND == 1 ? f[i1] : 1.f;
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        ox[x][0] = e0 * (ox[x][0] + ol[x][0]); ox[x][1] = e0 * (ox[x][1] + ol[x][1]);
        ox[x][2] = e1 * (ox[x][2] + ol[x][2]); ox[x][3] = e1 * (ox[x][3] + ol[x][3]);
      }
      for (int k0 = 0; k0 <= m0; k0 += 16) {     // o += P v
        uint32_t ph[4], pl[4], bv[4];
        const uint32_t at = b + L.p + oc_unit(m0 + (lane & 15), (k0 >> 3) + (lane >> 4));
        oc_ldsm4(ph, at);
        oc_ldsm4(pl, at + kPlane);
        oc_ldsm4t(bv, oc_b(sv, k0, n0, lane));
        oc_mman<2>(ox, ph, bv);
        oc_mman<2>(ox, pl, bv);
      }
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int cc = v0 + n0 + x * 8 + col;
        if (cc >= V) continue;
        if (i0 < n) *reinterpret_cast<float2*>(p.o + ((size_t)(t0 + i0) * p.H + h) * V + cc) = make_float2(ox[x][0], ox[x][1]);
        if (i1 < n) *reinterpret_cast<float2*>(p.o + ((size_t)(t0 + i1) * p.H + h) * V + cc) = make_float2(ox[x][2], ox[x][3]);
      }
    }
    if (whole || KIND == 1) __syncthreads();     // (the state operand is read, the weighted rows are there)
#pragma unroll
    for (int i = 0; i < MI; ++i) {               // the state
      const int piece = warp + 16 * i, d0 = (piece >> 1) * 16, c0 = (piece & 1) * 32;
      if (d0 >= D) continue;
      float f0, f1;
      if (KIND == 1) {
        f0 = f1 = f[kC - 1];
      } else {
        const float g0 = f[d0 + (lane >> 2)], g1 = f[d0 + (lane >> 2) + 8];
        total[i][0] += g0;
        total[i][1] += g1;
        f0 = exp2f(g0);
        f1 = exp2f(g1);
      }
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        hs[i][x][0] *= f0; hs[i][x][1] *= f0;
        hs[i][x][2] *= f1; hs[i][x][3] *= f1;
      }
      if (KIND == 1) total[i][0] += log2f(f0);
#pragma unroll
      for (int k0 = 0; k0 < kC; k0 += 16) {
        uint32_t kh[4], kl[4], bh[8], bl[8];
        oc_ldsm4t(kh, sk + krow + k0 * stride + d0 * 2);
        if (KIND == 0) oc_ldsm4t(kl, sk + plane + krow + k0 * stride + d0 * 2);
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          oc_ldsm4t(bh + 4 * x, oc_b(KIND == 1 ? base + L.w : sv, k0, c0 + x * 16, lane));
          if (KIND == 1) oc_ldsm4t(bl + 4 * x, oc_b(base + L.w + kPlane, k0, c0 + x * 16, lane));
        }
        oc_mman<4>(hs[i], kh, bh);
        if (KIND == 1) oc_mman<4>(hs[i], kh, bl);
        else oc_mman<4>(hs[i], kl, bh);
      }
    }
    if (whole) store_state();
    if (L.bufs == 1) {
      __syncthreads();
      fetch(c + 1);
    }
    oc_wait<0>();
    __syncthreads();
  }
  const size_t at = (size_t)(ws0 + seg) * p.H + h;
  float* to = last ? state : p.ws + at * size + v0;
  each_state([&](float& x, float& y, int d, int c) { *reinterpret_cast<float2*>(to + (size_t)d * V + c) = make_float2(x, y); });
  if (!last && !whole && blockIdx.x == 0 && (lane & 3) == 0) {
#pragma unroll
    for (int i = 0; i < MI; ++i) {
      const int piece = warp + 16 * i, d = (piece >> 1) * 16 + (lane >> 2);
      if ((piece & 1) || d >= D) continue;
      p.ws_decay[at * D + d] = total[i][0];
      p.ws_decay[at * D + d + 8] = KIND == 1 ? total[i][0] : total[i][1];
    }
  }
}

template <int KIND, int MI>
static cudaError_t launch_scan(const B200Outer& a, cudaStream_t stream) {
  const size_t smem = (size_t)scan_smem(KIND, a.D).total + 128;
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(outer_scan_kernel<KIND, MI>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
  const dim3 grid((a.V + kVs - 1) / kVs, a.H, a.rows.num_tiles);
  const cudaError_t e = launch_pdl(outer_scan_kernel<KIND, MI>, grid, dim3(kScanThreads), smem, stream, a, 0);
  if (e != cudaSuccess || !a.multi) return e;
  return launch_pdl(outer_scan_kernel<KIND, MI>, grid, dim3(kScanThreads), smem, stream, a, 1);
}

static size_t pairs_smem(const B200Outer* a) {
  return (a->kind == 0 ? (size_t)channel_smem(a->D, a->rank).total : (size_t)2 * kC * (a->D + 8) * 2) + 128;
}

}  // namespace b200

using namespace b200;

extern "C" {

// 1: the chunk kernels serve these sizes.
int b200_outer_fits(const B200Outer* a) {
  return outer_ok(a) && !a->f32 && a->D <= 256 && !(a->ld & 7) && !(a->kind == 0 && (a->lda1 & 7)) &&
         !(((uintptr_t)a->q | (uintptr_t)a->k | (uintptr_t)a->v | (uintptr_t)a->a1 | (uintptr_t)a->a2) & 15) &&
         pairs_smem(a) <= (a->kind == 0 ? 227 : 128) * 1024 && scan_smem(a->kind, a->D).total + 128 <= 227 * 1024;
}

// bf16 and fp32 workspace values (pairs, factors) of a chunk and state.
void b200_outer_workspace(int kind, int D, int* values) {
  values[0] = (int)pair_values(kind, D);
  values[1] = factor_values(kind, D);
}

// Leaves o of the portions in a->o and their states behind them.
int b200_outer_chunk(const B200Outer* a, cudaStream_t stream) {
  if (a->rows.num_prefills <= 0 || a->rows.num_tiles <= 0) return 0;
  if (!b200_outer_fits(a) || a->seg_tiles <= 0 || a->seg_tiles > 1 << 20 || (a->multi && (!a->ws || !a->ws_decay)) || !a->pairs ||
      !a->factors || (((uintptr_t)a->pairs | (uintptr_t)a->factors) & 15))
    return -1;
  if (a->H > 65535 || a->rows.num_tiles > 32767) return -4;
  const size_t smem = pairs_smem(a);
  cudaError_t e;
  if (a->kind == 0) {
    static PerDeviceOnce once;
    if (once.first()) cudaFuncSetAttribute(outer_pairs_channel_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    e = launch_pdl(outer_pairs_channel_kernel, dim3(a->H, 2 * a->rows.num_tiles), dim3(kPairThreads), smem, stream, *a);
  } else {
    static PerDeviceOnce once;
    if (once.first()) cudaFuncSetAttribute(outer_pairs_head_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
    const int slices = (a->H / a->G + kHeadsPerPair - 1) / kHeadsPerPair;
    e = launch_pdl(outer_pairs_head_kernel, dim3(a->G, 2 * a->rows.num_tiles, slices), dim3(kPairThreads), smem, stream, *a);
  }
  if (e != cudaSuccess) return -2;
  if (a->kind == 0) e = a->D <= 128 ? launch_scan<0, 1>(*a, stream) : launch_scan<0, 2>(*a, stream);
  else e = a->D <= 128 ? launch_scan<1, 1>(*a, stream) : launch_scan<1, 2>(*a, stream);
  return e == cudaSuccess ? 0 : -2;
}

}  // extern "C"
