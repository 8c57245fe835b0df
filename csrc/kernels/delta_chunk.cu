// Prompt portions of the gated delta rule (delta.cu) in chunks of 64 tokens, D <= 128, at fp32 accuracy on the
// tensor cores: every fp32 operand is kept as a bf16 pair (x = hi + lo) and a product is hi hi + hi lo + lo hi.
//
// With G_i the sum of the log decays up to token i inside a chunk and h the state before it, the writes u of a
// chunk solve  (I + A) u = r,  A[i, j] = beta_i e^(G_i - G_j) (k_i . k_j) for j < i,  r = beta (v - e^G (k h)), and
//   o = e^G (q h) + P u,  P[i, j] = e^(G_i - G_j) (q_i . k_j) for j <= i
//   h <- e^(G_last) h + k^T (e^(G_last - G) u)
// (the chunkwise form of the delta rule; Yang et al., "Gated Delta Networks", 2024).
//
//   delta_pairs_kernel   per (chunk, key head): k k^T and q k^T, then per head T = (I + A)^-1 by forward
//                        substitution in fp32, P, and the sums G; parallel over chunks
//   delta_scan_kernel    per (portion, head, 64 value columns): walks the chunks with h in registers
//                        (accumulators of the state update), three block barriers per chunk
//
// q and k rows of portions arrive as [hi (D) | lo (D)] bf16 pairs (b200_delta_prepare with ``split``). Rows past
// the end of a portion are zeros with beta = 0, g = 0, so they write nothing. T and P are lower triangular:
// of row block b (16 rows) only the first 16 (b + 1) columns exist.
#include "api.h"
#include "sm100.cuh"

namespace b200 {

typedef __nv_bfloat16 bf16;

static constexpr int kC = 64;                    // tokens per chunk
static constexpr int kVs = 64;                   // value columns per CTA of the scan
static constexpr int kThreads = 256;
static constexpr int kMat = kC * kC;             // one plane of T or P
static constexpr int kPlane = kC * 128;          // bytes of a 64 x 64 bf16 plane in shared memory

__device__ __forceinline__ void ldsm4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16(float* d, const uint32_t* a, const uint32_t* b) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
// d[4][4] += (ah + al)(bh + bl) for four 8-column tiles; b: 16 x 32, two x4 loads per plane.
__device__ __forceinline__ void mma_pairs(float (*d)[4], const uint32_t* ah, const uint32_t* al, const uint32_t* bh,
                                          const uint32_t* bl) {
#pragma unroll
  for (int n = 0; n < 4; ++n) mma16(d[n], ah, bh + 2 * n);
#pragma unroll
  for (int n = 0; n < 4; ++n) mma16(d[n], ah, bl + 2 * n);
#pragma unroll
  for (int n = 0; n < 4; ++n) mma16(d[n], al, bh + 2 * n);
}
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(x - h.x, y - h.y);
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool real) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(real ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// byte offset of 16-byte unit ``u`` of row ``r`` in a plane of 128-byte rows (units xored by the row)
__device__ __forceinline__ uint32_t unit(int r, int u) { return (uint32_t)(r * 128 + ((u ^ (r & 7)) << 4)); }
// the address a lane gives ldmatrix.trans for a 16 (k) x 16 (n) block of such a plane at (k0, n0)
__device__ __forceinline__ uint32_t b_addr(uint32_t base, int k0, int n0, int lane) {
  return base + unit(k0 + (lane & 15), (n0 >> 3) + (lane >> 4));
}

// K or Q rows [hi | lo] of a chunk to two planes of (D + 8)-wide rows
__device__ __forceinline__ void load_rows(uint32_t dst, const float* src, int t0, int len, int G, int g, int D, int tid) {
  const int u = D / 8, plane = kC * (D + 8) * 2;
  for (int x = tid; x < kC * 2 * u; x += kThreads) {
    const int r = x / (2 * u), c = x - r * 2 * u, lo = c >= u;
    const bool real = r < len;
    const bf16* s = reinterpret_cast<const bf16*>(src + ((size_t)(t0 + (real ? r : 0)) * G + g) * D) + c * 8;
    cp16(dst + lo * plane + r * (D + 8) * 2 + (c - lo * u) * 16, s, real);
  }
}
// the existing blocks of T or P
__device__ __forceinline__ void load_lower(uint32_t dst, const bf16* src, int tid) {
  for (int x = tid; x < 2 * kC * 8; x += kThreads) {
    const int p = x >> 9, r = (x >> 3) & 63, c = x & 7;
    if (c < 2 * (r / 16 + 1)) cp16(dst + p * kPlane + unit(r, c), src + p * kMat + r * kC + c * 8, true);
  }
}

struct DeltaChunkArgs {
  B200Delta p;
  bf16* tp;                // [chunks][H]: T hi | T lo | P hi | P lo
  float* gc;               // [chunks][H][64]
};

// ---------------------------------------------------------------------------------------------- pairs
// grid (2 per 128-row tile, G). Warp w owns rows 16 (w % 4) and columns 32 (w / 4) of both products.
__global__ void __launch_bounds__(kThreads) delta_pairs_kernel(DeltaChunkArgs a) {
  extern __shared__ uint8_t pair_raw[];
  const B200Delta& p = a.p;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(pair_raw) + 127) & ~uintptr_t(127));
  const int D = p.D, stride = (D + 8) * 2, plane = kC * stride, R = p.H / p.G;
  constexpr int kAt = 68;                        // row stride of the transposed A
  float* Ts = reinterpret_cast<float*>(smem);    // [2][64][64], over K and Q once their products are done
  const int kq_bytes = max(4 * plane, 2 * kMat * 4);
  float* At = reinterpret_cast<float*>(smem + kq_bytes);           // [2][64][kAt]
  float* sG = At + 2 * kC * kAt;                                   // [2][64]
  float* sB = sG + 2 * kC;                                         // [2][64]
  pdl_wait();
  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = blockIdx.y;
  const int tile = blockIdx.x >> 1, req = p.tile_req[tile], q0 = p.tile_q0[tile] + (blockIdx.x & 1) * kC;
  const int begin = p.q_start[req], len = min(kC, p.q_start[req + 1] - begin - q0);
  if (len <= 0 || p.slots[p.nd + req] < 0) return;
  const int t0 = p.nd + begin + q0;
  const uint32_t sk = smem_u32(smem), sq = sk + 2 * plane;
  load_rows(sk, p.k, t0, len, p.G, g, D, tid);
  load_rows(sq, p.q, t0, len, p.G, g, D, tid);
  cp_commit();
  cp_wait<0>();
  __syncthreads();
  const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 32, row = m0 + (lane >> 2);
  float kk[4][4], qk[4][4];
#pragma unroll
  for (int n = 0; n < 4; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) kk[n][e] = qk[n][e] = 0.f;
  if (n0 <= m0) {                                // (blocks above the diagonal are not needed)
    const uint32_t arow = (m0 + (lane & 15)) * stride + (lane >> 4) * 16;
    // B = K^T: the k index runs along K's rows, so no transpose: lanes give rows n, halves k
    const uint32_t brow = (n0 + (lane & 7) + ((lane >> 4) << 3)) * stride + ((lane >> 3) & 1) * 16;
    for (int k0 = 0; k0 < D; k0 += 16) {
      uint32_t kh[4], kl[4], qh[4], ql[4], bh[8], bl[8];
      ldsm4(kh, sk + arow + k0 * 2);
      ldsm4(kl, sk + plane + arow + k0 * 2);
      ldsm4(qh, sq + arow + k0 * 2);
      ldsm4(ql, sq + plane + arow + k0 * 2);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        ldsm4(bh + 4 * x, sk + brow + x * 16 * stride + k0 * 2);
        ldsm4(bl + 4 * x, sk + plane + brow + x * 16 * stride + k0 * 2);
      }
      mma_pairs(kk, kh, kl, bh, bl);
      mma_pairs(qk, qh, ql, bh, bl);
    }
  }
  for (int r0 = 0; r0 < R; r0 += 2) {
    const int nh = min(2, R - r0);
    __syncthreads();
    // sums of the log decays: warp w < nh scans head w
    if (warp < nh) {
      const int h = g * R + r0 + warp;
      float carry = 0.f;
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int i = x * 32 + lane;
        float v = i < len ? p.g[(size_t)(t0 + i) * p.H + h] : 0.f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float u = __shfl_up_sync(0xffffffffu, v, o);
          if (lane >= o) v += u;
        }
        v += carry;
        carry = __shfl_sync(0xffffffffu, v, 31);
        sG[warp * kC + i] = v;
        sB[warp * kC + i] = i < len ? p.beta[(size_t)(t0 + i) * p.H + h] : 0.f;
        a.gc[((size_t)blockIdx.x * p.H + h) * kC + i] = v;
      }
    }
    __syncthreads();
    if (n0 <= m0) {
      for (int x = 0; x < nh; ++x) {
        const float* G = sG + x * kC;
        bf16* P = a.tp + ((size_t)blockIdx.x * p.H + g * R + r0 + x) * 4 * kMat + 2 * kMat;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = row + half * 8;
          const float gi = G[i], bi = sB[x * kC + i];
#pragma unroll
          for (int n = 0; n < 4; ++n) {
            const int j = n0 + n * 8 + (lane & 3) * 2;
            if (j >= m0 + 16) continue;          // beyond the row block's columns
            const float e0 = j <= i ? expf(gi - G[j]) : 0.f, e1 = j + 1 <= i ? expf(gi - G[j + 1]) : 0.f;
            At[(x * kC + j) * kAt + i] = j < i ? bi * e0 * kk[n][half * 2] : 0.f;
            At[(x * kC + j + 1) * kAt + i] = j + 1 < i ? bi * e1 * kk[n][half * 2 + 1] : 0.f;
            uint32_t hi, lo;
            split_pair(e0 * qk[n][half * 2], e1 * qk[n][half * 2 + 1], hi, lo);
            *reinterpret_cast<uint32_t*>(P + i * kC + j) = hi;
            *reinterpret_cast<uint32_t*>(P + kMat + i * kC + j) = lo;
          }
        }
      }
    }
    __syncthreads();
    if (warp < 2 * nh) {
      // thread = one column of T; earlier rows of the column are its own, so no barrier is needed
      const int x = warp >> 1, c = tid & 63;
      const float* A = At + x * kC * kAt;
      float* T = Ts + x * kMat + c;
      bf16* out = a.tp + ((size_t)blockIdx.x * p.H + g * R + r0 + x) * 4 * kMat + c;
      for (int b = 0; b < 4; ++b) {
        float t[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) t[i] = b * 16 + i == c ? 1.f : 0.f;
        for (int j = 0; j < b * 16; ++j) {
          const float tj = T[j * kC];
          const float4* aj = reinterpret_cast<const float4*>(A + j * kAt + b * 16);
#pragma unroll
          for (int i4 = 0; i4 < 4; ++i4) {
            const float4 v = aj[i4];
            t[i4 * 4] -= v.x * tj; t[i4 * 4 + 1] -= v.y * tj; t[i4 * 4 + 2] -= v.z * tj; t[i4 * 4 + 3] -= v.w * tj;
          }
        }
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          const float* aj = A + (b * 16 + j) * kAt + b * 16;
#pragma unroll
          for (int i = j + 1; i < 16; ++i) t[i] -= aj[i] * t[j];
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int r = b * 16 + i;
          T[r * kC] = t[i];
          if (c < b * 16 + 16) {
            const bf16 hi = __float2bfloat16(t[i]);
            out[r * kC] = hi;
            out[kMat + r * kC] = __float2bfloat16(t[i] - __bfloat162float(hi));
          }
        }
      }
    }
  }
}

static size_t pairs_smem(int D) {
  const size_t kq = (size_t)4 * kC * (D + 8) * 2, ts = (size_t)2 * kMat * 4;
  return (kq > ts ? kq : ts) + (size_t)2 * kC * 68 * 4 + 4 * kC * 4 + 128;
}

// ----------------------------------------------------------------------------------------------- scan
struct ScanSmem { int k, q, h, t, p, r, u, w, total; };
__host__ __device__ inline ScanSmem scan_smem(int D) {
  ScanSmem s;
  const int rows = 2 * kC * (D + 8) * 2, mat = 2 * kPlane;
  int o = 0;
  s.h = o; o += 2 * D * 128;
  s.t = o; o += mat;
  s.p = o; o += mat;
  s.r = o; o += mat;
  s.u = o; o += mat;
  s.w = o; o += mat;
  s.k = o; o += 2 * rows;
  s.q = o; o += rows;
  s.total = o;
  return s;
}

// Warp w: rows 16 (w % 4), columns 32 (w / 4) of every 64 x 64 result; of the state, 16 x 32 pieces
// w, w + 8, ... (row block piece / 2, column half piece % 2), MI of them at most.
template <int MI>
__global__ void __launch_bounds__(kThreads, 1) delta_scan_kernel(DeltaChunkArgs a) {
  extern __shared__ uint8_t scan_raw[];
  const B200Delta& p = a.p;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(scan_raw) + 127) & ~uintptr_t(127));
  const int D = p.D, V = p.V, stride = (D + 8) * 2, plane = kC * stride, hplane = D * 128;
  const ScanSmem L = scan_smem(D);
  const uint32_t base = smem_u32(smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int v0 = blockIdx.x * kVs, h = blockIdx.y, req = blockIdx.z, g = h / (p.H / p.G);
  pdl_wait();
  pdl_launch_dependents();
  const int slot = p.slots[p.nd + req], begin = p.q_start[req], len = p.q_start[req + 1] - begin;
  if (len <= 0) return;
  const int chunks = (len + kC - 1) / kC, t_base = p.nd + begin;
  if (slot < 0) return;
  int first = 0;                                 // chunks of the portions ahead (two per 128-row tile)
  for (int i = lane; i < req; i += 32) first += (p.q_start[i + 1] - p.q_start[i] + 127) / 128 * 2;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) first += __shfl_xor_sync(0xffffffffu, first, o);
  const bool init = p.seq_lens[p.nd + req] > len;
  const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 32, col = (lane & 3) * 2;
  float* state = p.state + ((size_t)slot * p.H + h) * D * V + v0;
  float hs[MI][4][4];
#pragma unroll
  for (int i = 0; i < MI; ++i) {
    const int piece = warp + 8 * i, d0 = (piece >> 1) * 16 + (lane >> 2), c0 = (piece & 1) * 32 + col;
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int d = d0 + half * 8, c = c0 + n * 8;
        float2 x = make_float2(0.f, 0.f);
        if (init && d < D && v0 + c < V) x = *reinterpret_cast<const float2*>(state + (size_t)d * V + c);
        hs[i][n][half * 2] = x.x;
        hs[i][n][half * 2 + 1] = x.y;
      }
  }
  const bf16* tp = a.tp + ((size_t)first * p.H + h) * 4 * kMat;
  const size_t tp_step = (size_t)p.H * 4 * kMat;
  load_rows(base + L.k, p.k, t_base, min(kC, len), p.G, g, D, tid);
  load_rows(base + L.q, p.q, t_base, min(kC, len), p.G, g, D, tid);
  load_lower(base + L.t, tp, tid);
  cp_commit();

  const uint32_t arow = (m0 + (lane & 15)) * stride + (lane >> 4) * 16;
  const bf16* vp = reinterpret_cast<const bf16*>(p.v);
  for (int c = 0; c < chunks; ++c, tp += tp_step) {
    const int t0 = t_base + c * kC, n = min(kC, len - c * kC), i0 = m0 + (lane >> 2), i1 = i0 + 8;
    const int next = min(kC, len - (c + 1) * kC);
    const uint32_t sk = base + L.k + (c & 1) * 2 * plane, sq = base + L.q;
    // what the rows of this thread need: asked for ahead of the barrier
    const float* gc = a.gc + ((size_t)(first + c) * p.H + h) * kC;
    const float g0 = gc[i0], g1 = gc[i1], gl = gc[kC - 1];
    const float b0 = i0 < n ? p.beta[(size_t)(t0 + i0) * p.H + h] : 0.f, b1 = i1 < n ? p.beta[(size_t)(t0 + i1) * p.H + h] : 0.f;
    uint32_t vv[4][2];
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int cc = v0 + n0 + x * 8 + col;
      vv[x][0] = i0 < n && cc < V ? *reinterpret_cast<const uint32_t*>(vp + ((size_t)(t0 + i0) * p.H + h) * V + cc) : 0u;
      vv[x][1] = i1 < n && cc < V ? *reinterpret_cast<const uint32_t*>(vp + ((size_t)(t0 + i1) * p.H + h) * V + cc) : 0u;
    }
    // ---- the state as an operand
#pragma unroll
    for (int i = 0; i < MI; ++i) {
      const int piece = warp + 8 * i, d = (piece >> 1) * 16 + (lane >> 2);
      if (d >= D) continue;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int u = (piece & 1) * 4 + x;
        uint32_t hi, lo;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          split_pair(hs[i][x][half * 2], hs[i][x][half * 2 + 1], hi, lo);
          uint8_t* dst = smem + L.h + unit(d + half * 8, u) + col * 2;
          *reinterpret_cast<uint32_t*>(dst) = hi;
          *reinterpret_cast<uint32_t*>(dst + hplane) = lo;
        }
      }
    }
    cp_wait<0>();
    __syncthreads();
    load_lower(base + L.p, tp + 2 * kMat, tid);
    cp_commit();
    if (next > 0) load_rows(base + L.k + ((c + 1) & 1) * 2 * plane, p.k, t0 + kC, next, p.G, g, D, tid);
    cp_commit();
    // ---- k h and q h
    float kx[4][4], ox[4][4];
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) kx[x][e] = ox[x][e] = 0.f;
#pragma unroll 2
    for (int k0 = 0; k0 < D; k0 += 16) {
      uint32_t kh[4], kl[4], qh[4], ql[4], bh[8], bl[8];
      ldsm4(kh, sk + arow + k0 * 2);
      ldsm4(kl, sk + plane + arow + k0 * 2);
      ldsm4(qh, sq + arow + k0 * 2);
      ldsm4(ql, sq + plane + arow + k0 * 2);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        ldsm4t(bh + 4 * x, b_addr(base + L.h, k0, n0 + x * 16, lane));
        ldsm4t(bl + 4 * x, b_addr(base + L.h + hplane, k0, n0 + x * 16, lane));
      }
      mma_pairs(kx, kh, kl, bh, bl);
      mma_pairs(ox, qh, ql, bh, bl);
    }
    const float e0 = expf(g0), e1 = expf(g1);
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const float2 w0 = unpack_bf16x2(vv[x][0]), w1 = unpack_bf16x2(vv[x][1]);
      uint32_t hi, lo;
      uint8_t* dst = smem + L.r + unit(i0, n0 / 8 + x) + col * 2;
      split_pair(b0 * (w0.x - e0 * kx[x][0]), b0 * (w0.y - e0 * kx[x][1]), hi, lo);
      *reinterpret_cast<uint32_t*>(dst) = hi;
      *reinterpret_cast<uint32_t*>(dst + kPlane) = lo;
      dst = smem + L.r + unit(i1, n0 / 8 + x) + col * 2;
      split_pair(b1 * (w1.x - e1 * kx[x][2]), b1 * (w1.y - e1 * kx[x][3]), hi, lo);
      *reinterpret_cast<uint32_t*>(dst) = hi;
      *reinterpret_cast<uint32_t*>(dst + kPlane) = lo;
      ox[x][0] *= e0; ox[x][1] *= e0; ox[x][2] *= e1; ox[x][3] *= e1;
    }
    __syncthreads();
    if (next > 0) load_rows(sq, p.q, t0 + kC, next, p.G, g, D, tid);
    cp_commit();
    // ---- u = T r
    float ux[4][4];
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) ux[x][e] = 0.f;
    for (int k0 = 0; k0 <= m0; k0 += 16) {
      uint32_t th[4], tl[4], bh[8], bl[8];
      const uint32_t at = base + L.t + unit(m0 + (lane & 15), (k0 >> 3) + (lane >> 4));
      ldsm4(th, at);
      ldsm4(tl, at + kPlane);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        ldsm4t(bh + 4 * x, b_addr(base + L.r, k0, n0 + x * 16, lane));
        ldsm4t(bl + 4 * x, b_addr(base + L.r + kPlane, k0, n0 + x * 16, lane));
      }
      mma_pairs(ux, th, tl, bh, bl);
    }
    const float f0 = expf(gl - g0), f1 = expf(gl - g1);
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      uint32_t hi, lo;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const uint32_t off = unit(half ? i1 : i0, n0 / 8 + x) + col * 2;
        const float f = half ? f1 : f0, y0 = ux[x][half * 2], y1 = ux[x][half * 2 + 1];
        split_pair(y0, y1, hi, lo);
        *reinterpret_cast<uint32_t*>(smem + L.u + off) = hi;
        *reinterpret_cast<uint32_t*>(smem + L.u + kPlane + off) = lo;
        split_pair(f * y0, f * y1, hi, lo);
        *reinterpret_cast<uint32_t*>(smem + L.w + off) = hi;
        *reinterpret_cast<uint32_t*>(smem + L.w + kPlane + off) = lo;
      }
    }
    cp_wait<2>();                                // P has arrived (the next k and q may still be on the way)
    __syncthreads();
    if (next > 0) load_lower(base + L.t, tp + tp_step, tid);
    cp_commit();
    // ---- o += P u
    for (int k0 = 0; k0 <= m0; k0 += 16) {
      uint32_t ph[4], pl[4], bh[8], bl[8];
      const uint32_t at = base + L.p + unit(m0 + (lane & 15), (k0 >> 3) + (lane >> 4));
      ldsm4(ph, at);
      ldsm4(pl, at + kPlane);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        ldsm4t(bh + 4 * x, b_addr(base + L.u, k0, n0 + x * 16, lane));
        ldsm4t(bl + 4 * x, b_addr(base + L.u + kPlane, k0, n0 + x * 16, lane));
      }
      mma_pairs(ox, ph, pl, bh, bl);
    }
    // ---- h <- e^(G_last) h + k^T w
    const float decay = expf(gl);
    const uint32_t krow = ((lane & 7) + (lane >> 4) * 8) * stride + ((lane >> 3) & 1) * 16;
#pragma unroll
    for (int i = 0; i < MI; ++i) {
      const int piece = warp + 8 * i, d0 = (piece >> 1) * 16, c0 = (piece & 1) * 32;
      if (d0 >= D) continue;
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) hs[i][x][e] *= decay;
#pragma unroll
      for (int k0 = 0; k0 < kC; k0 += 16) {
        uint32_t kh[4], kl[4], bh[8], bl[8];
        ldsm4t(kh, sk + krow + k0 * stride + d0 * 2);
        ldsm4t(kl, sk + plane + krow + k0 * stride + d0 * 2);
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          ldsm4t(bh + 4 * x, b_addr(base + L.w, k0, c0 + x * 16, lane));
          ldsm4t(bl + 4 * x, b_addr(base + L.w + kPlane, k0, c0 + x * 16, lane));
        }
        mma_pairs(hs[i], kh, kl, bh, bl);
      }
    }
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int cc = v0 + n0 + x * 8 + col;
      if (cc >= V) continue;
      if (i0 < n) *reinterpret_cast<float2*>(p.o + ((size_t)(t0 + i0) * p.H + h) * V + cc) = make_float2(ox[x][0], ox[x][1]);
      if (i1 < n) *reinterpret_cast<float2*>(p.o + ((size_t)(t0 + i1) * p.H + h) * V + cc) = make_float2(ox[x][2], ox[x][3]);
    }
  }
  cp_wait<0>();
#pragma unroll
  for (int i = 0; i < MI; ++i) {
    const int piece = warp + 8 * i, d0 = (piece >> 1) * 16 + (lane >> 2), c0 = (piece & 1) * 32 + col;
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int d = d0 + half * 8, c = c0 + n * 8;
        if (d < D && v0 + c < V)
          *reinterpret_cast<float2*>(state + (size_t)d * V + c) = make_float2(hs[i][n][half * 2], hs[i][n][half * 2 + 1]);
      }
  }
}

template <int MI>
static cudaError_t launch_scan(const DeltaChunkArgs& a, cudaStream_t stream) {
  const size_t smem = (size_t)scan_smem(a.p.D).total + 128;
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(delta_scan_kernel<MI>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
  return launch_pdl(delta_scan_kernel<MI>, dim3((a.p.V + kVs - 1) / kVs, a.p.H, a.p.num_prefills), dim3(kThreads), smem,
                    stream, a);
}

}  // namespace b200

using namespace b200;

extern "C" {

// 1: the chunk kernels serve these sizes.
int b200_delta_chunk_fits(const B200Delta* a) {
  return !a->f32 && a->D > 0 && a->D <= 128 && !(a->D & 15) && a->V > 0 && !(a->V & 15) &&
         scan_smem(a->D).total + 128 <= 227 * 1024;
}

// tp: bf16 [2 num_tiles][H][4][64][64], gc: fp32 [2 num_tiles][H][64]. Leaves o of the portions in a->o.
int b200_delta_chunk(const B200Delta* a, void* tp, void* gc, cudaStream_t stream) {
  if (a->num_prefills <= 0 || a->num_tiles <= 0) return 0;
  if (!b200_delta_chunk_fits(a) || !a->split || a->G <= 0 || a->H % a->G || !tp || !gc) return -1;
  if (a->H > 65535 || a->num_prefills > 65535) return -4;
  const DeltaChunkArgs x{*a, (bf16*)tp, (float*)gc};
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(delta_pairs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)pairs_smem(128));
  if (launch_pdl(delta_pairs_kernel, dim3(2 * a->num_tiles, a->G), dim3(kThreads), pairs_smem(a->D), stream, x) != cudaSuccess)
    return -2;
  const int mi = (a->D + 63) / 64;
  return (mi == 1 ? launch_scan<1>(x, stream) : launch_scan<2>(x, stream)) == cudaSuccess ? 0 : -2;
}

}  // extern "C"
