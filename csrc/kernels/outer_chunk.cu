// Prompt portions of the recurrences over outer products (outer.cu) in chunks of 64 tokens, D <= 256, at fp32 accuracy
// on the tensor cores: fp32 operands are kept as bf16 pairs (x = hi + lo, products hi hi + hi lo + lo hi); operands
// that arrive as bf16 are used as they are.
//
// With G_i the sum of the log decays up to token i inside a chunk (per key channel, or one per head) and S the state
// before it,
//   o_i = (q_i e^(G_i))^T S + sum_{j <= i} P_ij v_j,   P_ij = sum_d q_id k_jd e^(G_id - G_jd)
//   S <- e^(G_last) S + sum_j (k_j e^(G_last - G_j)) v_j^T
// Decay per head (kind 1): P is (q k^T) times e^(G_i - G_j) dt_j, and dt_j e^(G_last - G_j) goes with v_j.
// Decay per channel (kind 0): with q' = q e^G and k' = k e^-G, P = q' k'^T and S <- e^(G_last) (S + k'^T v). e^-G stays
// below e^60 as long as no channel fades by more than that inside the chunk; where one does, the chunk is walked in
// steps of 16 tokens, and where even those are too far apart, token by token (a single token's decay is cut off at
// e^-60). (The chunkwise forms; Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training";
// Dao and Gu, "Transformers are SSMs".)
//
// grid (64-wide slices of the value columns, H, 128-row tiles). A CTA walks one segment of a portion: ``seg_tiles`` tiles
// from its own on (other tiles' CTAs return), the state in registers as accumulators of its update. A portion of several
// segments takes two launches. The first runs segment 0 and leaves the state behind it, and for the segments in between
// the state they would leave if they started from zero, with their decay. The second runs the segments from 1 on, each from
// the state that it puts together from those. Only the last one writes the slot's state, which nobody reads any more.
#include "api.h"
#include "sm100.cuh"

namespace b200 {

typedef __nv_bfloat16 bf16;
bool outer_ok(const B200Outer* a);

static constexpr int kC = 64;                    // tokens per chunk
static constexpr int kVs = 64;                   // value columns per CTA
static constexpr int kThreads = 256;
static constexpr int kPlane = kC * 128;          // bytes of a 64 x 64 bf16 plane
static constexpr float kMostDecay = 60.f;

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
// d[4][4] += a b for four 8-column tiles; b: 16 x 32, two x4 loads
__device__ __forceinline__ void oc_mma4(float (*d)[4], const uint32_t* a, const uint32_t* b) {
#pragma unroll
  for (int n = 0; n < 4; ++n) oc_mma(d[n], a, b + 2 * n);
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
__device__ __forceinline__ float oc_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// byte offset of 16-byte unit ``u`` of row ``r`` in a plane of 128-byte rows (units xored by the row)
__device__ __forceinline__ uint32_t oc_unit(int r, int u) { return (uint32_t)(r * 128 + ((u ^ (r & 7)) << 4)); }
// the address a lane gives ldmatrix.trans for a 16 (k) x 16 (n) block of such a plane at (k0, n0)
__device__ __forceinline__ uint32_t oc_b(uint32_t base, int k0, int n0, int lane) {
  return base + oc_unit(k0 + (lane & 15), (n0 >> 3) + (lane >> 4));
}

struct ChunkSmem { int q, k, s, p, v, w, a1, f, total, bufs; };
__host__ __device__ inline ChunkSmem chunk_smem(int kind, int D, int rank) {
  ChunkSmem m;
  const int rows = kC * (D + 8) * 2;             // a plane of q or k rows
  int o = 0;
  m.bufs = kind == 0 || D <= 128 ? 2 : 1;        // buffers of what arrives ahead
  m.s = o; o += 2 * D * 128;
  m.q = o; o += kind == 0 ? 2 * rows : m.bufs * rows;
  m.k = o; o += kind == 0 ? 2 * rows : m.bufs * rows;
  if (kind == 0 && D > 128) m.p = m.q;           // (over q', once the products with it are done)
  else { m.p = o; o += 2 * kPlane; }
  m.v = o; o += m.bufs * kPlane;
  m.w = o; o += kind == 1 ? 2 * kPlane : 0;
  m.a1 = o; o += kind == 0 ? 2 * kC * (rank + 8) * 2 : 0;
  m.f = o; o += kind == 0 ? D * 4 : 2 * 2 * kC * 4;      // e^(G_last) per channel, or two buffers of G and dt
  m.total = o;
  return m;
}

// KIND 0: decay per key channel, 1: per head. MI: 16 x 32 pieces of the state per warp (D <= 64 MI).
// Warp w: rows 16 (w % 4), columns 32 (w / 4) of every 64 x 64 result; of the state, pieces w, w + 8, ... (row block
// piece / 2, column half piece % 2); of q' and k', the 16-channel strips w, w + 8, ...
template <int KIND, int MI>
__global__ void __launch_bounds__(kThreads, 1) outer_chunk_kernel(B200Outer p, int phase) {
  extern __shared__ uint8_t chunk_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(chunk_raw) + 127) & ~uintptr_t(127));
  const int D = p.D, V = p.V, stride = (D + 8) * 2, plane = kC * stride, splane = D * 128;
  const ChunkSmem L = chunk_smem(KIND, D, p.rank);
  const uint32_t base = smem_u32(smem);
  float* sf = reinterpret_cast<float*>(smem + L.f);
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
  const bool init = R.seq_lens[R.nd + req] > len;
  const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 32, col = (lane & 3) * 2;
  const size_t size = (size_t)D * V;
  float* state = p.state + ((size_t)slot * p.H + h) * size + v0;
  float hs[MI][4][4];
  float total[MI][2];                            // decay of the rows of this thread's pieces since the segment's start (log)
  auto each_state = [&](auto f) {                // f(piece values, row, column) for pairs of columns
#pragma unroll
    for (int i = 0; i < MI; ++i) {
      const int piece = warp + 8 * i, d0 = (piece >> 1) * 16 + (lane >> 2), c0 = (piece & 1) * 32 + col;
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
        const float f = i == 0 ? 0.f : expf(w[d]);
        x = fmaf(f, x, u.x);
        y = fmaf(f, y, u.y);
      });
    }
  }

  const bf16* gq = reinterpret_cast<const bf16*>(p.q) + (size_t)g * D;
  const bf16* gk = reinterpret_cast<const bf16*>(p.k) + (size_t)g * D;
  const bf16* gv = reinterpret_cast<const bf16*>(p.v) + (size_t)h * V + v0;
  const int rank = p.rank, astride = (rank + 8) * 2;
  // what arrives by cp.async: v and the decay's factors (kind 0), v, q and k rows (kind 1)
  auto fetch = [&](int c) {
    if (c < chunks) {
      const int t0 = t_base + c * kC, n = min(kC, rows - c * kC), b = c % L.bufs;
      for (int x = tid; x < kC * 8; x += kThreads) {
        const int r = x >> 3, u = x & 7;
        const bool real = r < n && v0 + u * 8 < V;
        oc_cp16(base + L.v + b * kPlane + oc_unit(r, u), real ? gv + (size_t)(t0 + r) * p.ld + u * 8 : gv, real);
      }
      if (KIND == 0) {
        const int units = rank / 8;
        const bf16* a1 = reinterpret_cast<const bf16*>(p.a1);
        for (int x = tid; x < kC * units; x += kThreads) {
          const int r = x / units, u = x - r * units;
          oc_cp16(base + L.a1 + b * kC * astride + r * astride + u * 16, a1 + (size_t)(t0 + (r < n ? r : 0)) * p.lda1 + u * 8, r < n);
        }
      } else {
        const int units = D / 8;
        for (int x = tid; x < kC * units; x += kThreads) {
          const int r = x / units, u = x - r * units;
          const bool real = r < n;
          const size_t at = (size_t)(t0 + (real ? r : 0)) * p.ld + u * 8;
          if (whole) oc_cp16(base + L.q + b * plane + r * stride + u * 16, gq + at, real);
          oc_cp16(base + L.k + b * plane + r * stride + u * 16, gk + at, real);
        }
      }
    }
    oc_commit();
  };
  fetch(0);

  // kind 0: q' and k' of rows [lo, hi) of the chunk (the others become zeros) and e^(G) of the last of them; returns
  // whether a channel fades too far over all of them (1), over one of the blocks of 16 (2)
  auto scaled = [&](int c, int lo, int hi) {
    const int t0 = t_base + c * kC, b = c % L.bufs;
    int far = 0;
    for (int strip = warp; strip < D / 16; strip += 8) {
      const int cb = strip * 16 + col;           // channels cb + 8 nt, cb + 8 nt + 1
      uint32_t qv[4][2][2], kv[4][2][2];
#pragma unroll
      for (int mb = 0; mb < 4; ++mb)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = mb * 16 + half * 8 + (lane >> 2);
          const bool real = r >= lo && r < hi;
          const size_t at = (size_t)(t0 + r) * p.ld + cb;
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            kv[mb][half][nt] = real ? *reinterpret_cast<const uint32_t*>(gk + at + nt * 8) : 0u;
            qv[mb][half][nt] = real && whole ? *reinterpret_cast<const uint32_t*>(gq + at + nt * 8) : 0u;
          }
        }
      float z[4][2][4];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        const float2 bias = *reinterpret_cast<const float2*>(p.a2b + (size_t)h * D + cb + nt * 8);
#pragma unroll
        for (int mb = 0; mb < 4; ++mb) { z[mb][nt][0] = z[mb][nt][2] = bias.x; z[mb][nt][1] = z[mb][nt][3] = bias.y; }
      }
      const bf16* a2 = reinterpret_cast<const bf16*>(p.a2) + ((size_t)h * D + strip * 16 + (lane >> 2)) * rank + col;
      for (int k0 = 0; k0 < rank; k0 += 16) {
        uint32_t w[2][2];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e) w[nt][e] = *reinterpret_cast<const uint32_t*>(a2 + (size_t)nt * 8 * rank + k0 + e * 8);
#pragma unroll
        for (int mb = 0; mb < 4; ++mb) {
          uint32_t a[4];
          oc_ldsm4(a, base + L.a1 + b * kC * astride + (mb * 16 + (lane & 15)) * astride + (lane >> 4) * 16 + k0 * 2);
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) oc_mma(z[mb][nt], a, w[nt]);
        }
      }
      // log decays, then their sums down the rows (eight lanes, four apart, hold consecutive rows)
      float carry[2][2] = {{0.f, 0.f}, {0.f, 0.f}};
#pragma unroll
      for (int mb = 0; mb < 4; ++mb) {
        float before[2][2];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) { before[nt][0] = carry[nt][0]; before[nt][1] = carry[nt][1]; }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = mb * 16 + half * 8 + (lane >> 2);
          const bool real = r >= lo && r < hi;
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              float x = z[mb][nt][half * 2 + e];
              x = real ? fmaxf(-oc_softplus(-x) * p.inv_tau, -kMostDecay) : 0.f;
#pragma unroll
              for (int o = 4; o < 32; o <<= 1) {
                const float y = __shfl_up_sync(0xffffffffu, x, o);
                if (lane >= o) x += y;
              }
              x += carry[nt][e];
              carry[nt][e] = __shfl_sync(0xffffffffu, x, 28 + (lane & 3));
              z[mb][nt][half * 2 + e] = x;
            }
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e)
            if (carry[nt][e] - before[nt][e] < -kMostDecay) far |= 2;
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          if (carry[nt][e] < -kMostDecay) far |= 1;
          if (lane < 4) sf[cb + nt * 8 + e] = carry[nt][e];
        }
#pragma unroll
        for (int mb = 0; mb < 4; ++mb)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int r = mb * 16 + half * 8 + (lane >> 2);
            const float g0 = z[mb][nt][half * 2], g1 = z[mb][nt][half * 2 + 1];
            const float2 kk = unpack_bf16x2(kv[mb][half][nt]);
            uint8_t* dst = smem + r * stride + (cb + nt * 8) * 2;
            uint32_t hi2, lo2;
            oc_split(kk.x * expf(-g0), kk.y * expf(-g1), hi2, lo2);
            *reinterpret_cast<uint32_t*>(dst + L.k) = hi2;
            *reinterpret_cast<uint32_t*>(dst + L.k + plane) = lo2;
            if (whole) {
              const float2 qq = unpack_bf16x2(qv[mb][half][nt]);
              oc_split(p.q_scale * qq.x * expf(g0), p.q_scale * qq.y * expf(g1), hi2, lo2);
              *reinterpret_cast<uint32_t*>(dst + L.q) = hi2;
              *reinterpret_cast<uint32_t*>(dst + L.q + plane) = lo2;
            }
          }
      }
    }
    return far;
  };
  // kind 1: sums of the log decays and step sizes of a chunk (warp 0)
  auto steps = [&](int c) {
    const int t0 = t_base + c * kC, n = min(kC, rows - c * kC);
    float* f = sf + (c & 1) * 2 * kC;
    float carry = 0.f;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int i = x * 32 + lane;
      float dt = 0.f;
      if (i < n) dt = oc_softplus(__bfloat162float(reinterpret_cast<const bf16*>(p.dt)[(size_t)(t0 + i) * p.lddt + h]) + p.dt_bias[h]);
      float s = -p.A[h] * dt;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += y;
      }
      s += carry;
      carry = __shfl_sync(0xffffffffu, s, 31);
      f[i] = s;
      f[kC + i] = dt;
    }
  };
  auto store_state = [&]() {                     // the state as an operand
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
          oc_split(hs[i][x][half * 2], hs[i][x][half * 2 + 1], hi, lo);
          uint8_t* dst = smem + L.s + oc_unit(d + half * 8, u) + col * 2;
          *reinterpret_cast<uint32_t*>(dst) = hi;
          *reinterpret_cast<uint32_t*>(dst + splane) = lo;
        }
      }
    }
  };
  const uint32_t arow = (m0 + (lane & 15)) * stride + (lane >> 4) * 16;
  // B = K^T: the k index runs along K's rows, so no transpose: lanes give rows n, halves k
  const uint32_t brow = (n0 + (lane & 7) + ((lane >> 4) << 3)) * stride + ((lane >> 3) & 1) * 16;
  const uint32_t krow = ((lane & 7) + (lane >> 4) * 8) * stride + ((lane >> 3) & 1) * 16;
  const int i0 = m0 + (lane >> 2), i1 = i0 + 8;

  // Outputs and state of the rows that q', k' (kind 0) or the chunk's buffers hold; barriers: everything it reads is there.
  auto advance = [&](int c, float (*ox)[4]) {
    const int b = c % L.bufs;
    const uint32_t sq = base + L.q + (KIND == 1 ? b * plane : 0), sk = base + L.k + (KIND == 1 ? b * plane : 0);
    const uint32_t sv = base + L.v + b * kPlane;
    const float* f = sf + (KIND == 1 ? (c & 1) * 2 * kC : 0);
    if (KIND == 1) {                             // v rows with their weights, as pairs
      const float gl = f[kC - 1];
      for (int x = tid; x < kC * 32; x += kThreads) {
        const int r = x >> 5, cc = (x & 31) * 2;
        const uint32_t off = oc_unit(r, cc >> 3) + (cc & 7) * 2;
        const float2 y = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(smem + L.v + b * kPlane + off));
        const float w = f[kC + r] * expf(gl - f[r]);
        uint32_t hi, lo;
        oc_split(w * y.x, w * y.y, hi, lo);
        *reinterpret_cast<uint32_t*>(smem + L.w + off) = hi;
        *reinterpret_cast<uint32_t*>(smem + L.w + kPlane + off) = lo;
      }
    }
    if (whole) {
      float px[4][4], sx[4][4];
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) px[x][e] = sx[x][e] = 0.f;
      const bool lower = n0 <= m0;               // (blocks above the diagonal are not needed)
#pragma unroll 2
      for (int k0 = 0; k0 < D; k0 += 16) {
        uint32_t qh[4], ql[4], bh[8], bl[8];
        oc_ldsm4(qh, sq + arow + k0 * 2);
        if (KIND == 0) oc_ldsm4(ql, sq + plane + arow + k0 * 2);
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          oc_ldsm4t(bh + 4 * x, oc_b(base + L.s, k0, n0 + x * 16, lane));
          oc_ldsm4t(bl + 4 * x, oc_b(base + L.s + splane, k0, n0 + x * 16, lane));
        }
        oc_mma4(sx, qh, bh);
        oc_mma4(sx, qh, bl);
        if (KIND == 0) oc_mma4(sx, ql, bh);
        if (lower) {
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            oc_ldsm4(bh + 4 * x, sk + brow + x * 16 * stride + k0 * 2);
            if (KIND == 0) oc_ldsm4(bl + 4 * x, sk + plane + brow + x * 16 * stride + k0 * 2);
          }
          oc_mma4(px, qh, bh);
          if (KIND == 0) {
            oc_mma4(px, qh, bl);
            oc_mma4(px, ql, bh);
          }
        }
      }
      if (KIND == 0 && D > 128) __syncthreads(); // (P lies over q')
      const float e0 = KIND == 1 ? expf(f[i0]) : 1.f, e1 = KIND == 1 ? expf(f[i1]) : 1.f;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        ox[x][0] = fmaf(e0, sx[x][0], ox[x][0]); ox[x][1] = fmaf(e0, sx[x][1], ox[x][1]);
        ox[x][2] = fmaf(e1, sx[x][2], ox[x][2]); ox[x][3] = fmaf(e1, sx[x][3], ox[x][3]);
        const int j = n0 + x * 8 + col;
        if (!lower || j >= m0 + 16) continue;    // (beyond the row block's columns)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = half ? i1 : i0;
          float y0 = px[x][half * 2], y1 = px[x][half * 2 + 1];
          if (KIND == 1) {
            y0 = j <= i ? y0 * expf(f[i] - f[j]) * f[kC + j] : 0.f;
            y1 = j + 1 <= i ? y1 * expf(f[i] - f[j + 1]) * f[kC + j + 1] : 0.f;
          } else {
            y0 = j <= i ? y0 : 0.f;
            y1 = j + 1 <= i ? y1 : 0.f;
          }
          uint32_t hi, lo;
          oc_split(y0, y1, hi, lo);
          uint8_t* dst = smem + L.p + oc_unit(i, j >> 3) + col * 2;
          *reinterpret_cast<uint32_t*>(dst) = hi;
          *reinterpret_cast<uint32_t*>(dst + kPlane) = lo;
        }
      }
    }
    if (whole || KIND == 1) __syncthreads();
    if (whole) {
      for (int k0 = 0; k0 <= m0; k0 += 16) {     // o += P v
        uint32_t ph[4], pl[4], bv[8];
        const uint32_t at = base + L.p + oc_unit(m0 + (lane & 15), (k0 >> 3) + (lane >> 4));
        oc_ldsm4(ph, at);
        oc_ldsm4(pl, at + kPlane);
#pragma unroll
        for (int x = 0; x < 2; ++x) oc_ldsm4t(bv + 4 * x, oc_b(sv, k0, n0 + x * 16, lane));
        oc_mma4(ox, ph, bv);
        oc_mma4(ox, pl, bv);
      }
    }
#pragma unroll
    for (int i = 0; i < MI; ++i) {               // the state
      const int piece = warp + 8 * i, d0 = (piece >> 1) * 16, c0 = (piece & 1) * 32;
      if (d0 >= D) continue;
      float f0, f1;
      if (KIND == 1) {
        const float gl = f[kC - 1];
        total[i][0] += gl;
        f0 = expf(gl);
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
          for (int e = 0; e < 4; ++e) hs[i][x][e] *= f0;
      } else {
        const float g0 = f[d0 + (lane >> 2)], g1 = f[d0 + (lane >> 2) + 8];
        total[i][0] += g0;
        total[i][1] += g1;
        f0 = expf(g0);
        f1 = expf(g1);
      }
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
        oc_mma4(hs[i], kh, bh);
        if (KIND == 1) oc_mma4(hs[i], kh, bl);
        else oc_mma4(hs[i], kl, bh);
      }
      if (KIND == 0) {
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          hs[i][x][0] *= f0; hs[i][x][1] *= f0;
          hs[i][x][2] *= f1; hs[i][x][3] *= f1;
        }
      }
    }
  };

  for (int c = 0; c < chunks; ++c) {
    const int t0 = t_base + c * kC, n = min(kC, rows - c * kC);
    float ox[4][4];
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) ox[x][e] = 0.f;
    if (KIND == 0) {
      oc_wait<0>();
      __syncthreads();                           // v and the factors are there, q' and k' of the last chunk done with
      fetch(c + 1);
      const int far = scaled(c, 0, n);
      if (whole) store_state();
      if (!__syncthreads_or(far)) {
        advance(c, ox);
      } else {
        const int unit = __syncthreads_or(far & 2) ? 1 : 16;
        for (int lo = 0; lo < n; lo += unit) {
          __syncthreads();
          scaled(c, lo, min(lo + unit, n));
          if (whole) store_state();
          __syncthreads();
          advance(c, ox);
        }
      }
    } else {
      if (warp == 0) steps(c);
      if (whole) store_state();
      oc_wait<0>();
      __syncthreads();
      if (L.bufs == 2) fetch(c + 1);
      advance(c, ox);
      if (L.bufs == 1) {
        __syncthreads();
        fetch(c + 1);
      }
    }
    if (whole) {
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int cc = v0 + n0 + x * 8 + col;
        if (cc >= V) continue;
        if (i0 < n) *reinterpret_cast<float2*>(p.o + ((size_t)(t0 + i0) * p.H + h) * V + cc) = make_float2(ox[x][0], ox[x][1]);
        if (i1 < n) *reinterpret_cast<float2*>(p.o + ((size_t)(t0 + i1) * p.H + h) * V + cc) = make_float2(ox[x][2], ox[x][3]);
      }
    }
  }
  oc_wait<0>();
  const size_t at = (size_t)(ws0 + seg) * p.H + h;
  float* to = last ? state : p.ws + at * size + v0;
  each_state([&](float& x, float& y, int d, int c) { *reinterpret_cast<float2*>(to + (size_t)d * V + c) = make_float2(x, y); });
  if (!last && !whole && blockIdx.x == 0 && (lane & 3) == 0) {
#pragma unroll
    for (int i = 0; i < MI; ++i) {
      const int piece = warp + 8 * i, d = (piece >> 1) * 16 + (lane >> 2);
      if ((piece & 1) || d >= D) continue;
      p.ws_decay[at * D + d] = total[i][0];
      p.ws_decay[at * D + d + 8] = KIND == 1 ? total[i][0] : total[i][1];
    }
  }
}

template <int KIND, int MI>
static cudaError_t launch_chunks(const B200Outer& a, cudaStream_t stream) {
  const size_t smem = (size_t)chunk_smem(KIND, a.D, a.rank).total + 128;
  static PerDeviceOnce once;
  if (once.first())
    cudaFuncSetAttribute(outer_chunk_kernel<KIND, MI>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
  const dim3 grid((a.V + kVs - 1) / kVs, a.H, a.rows.num_tiles);
  const cudaError_t e = launch_pdl(outer_chunk_kernel<KIND, MI>, grid, dim3(kThreads), smem, stream, a, 0);
  if (e != cudaSuccess || !a.multi) return e;
  return launch_pdl(outer_chunk_kernel<KIND, MI>, grid, dim3(kThreads), smem, stream, a, 1);
}

}  // namespace b200

using namespace b200;

extern "C" {

// 1: the chunk kernel serves these sizes.
int b200_outer_fits(const B200Outer* a) {
  return outer_ok(a) && !a->f32 && a->D <= 256 && !(a->ld & 7) && !(a->kind == 0 && (a->lda1 & 7)) &&
         !(((uintptr_t)a->q | (uintptr_t)a->k | (uintptr_t)a->v | (uintptr_t)a->a1 | (uintptr_t)a->a2) & 15) &&
         chunk_smem(a->kind, a->D, a->rank).total + 128 <= 227 * 1024;
}

// Leaves o of the portions in a->o and their states behind them.
int b200_outer_chunk(const B200Outer* a, cudaStream_t stream) {
  if (a->rows.num_prefills <= 0 || a->rows.num_tiles <= 0) return 0;
  if (!b200_outer_fits(a) || a->seg_tiles <= 0 || a->seg_tiles > 1 << 20 || (a->multi && (!a->ws || !a->ws_decay))) return -1;
  if (a->H > 65535 || a->rows.num_tiles > 65535) return -4;
  const int mi = a->D <= 64 ? 1 : a->D <= 128 ? 2 : 4;
  cudaError_t e;
  if (a->kind == 0) e = mi == 1 ? launch_chunks<0, 1>(*a, stream) : mi == 2 ? launch_chunks<0, 2>(*a, stream) : launch_chunks<0, 4>(*a, stream);
  else e = mi == 1 ? launch_chunks<1, 1>(*a, stream) : mi == 2 ? launch_chunks<1, 2>(*a, stream) : launch_chunks<1, 4>(*a, stream);
  return e == cudaSuccess ? 0 : -2;
}

}  // extern "C"
