// Short causal convolutions and the real-gated linear recurrent unit with per-layer sizes; everything that
// enters the recurrence in fp32.
//
//   short_conv_kernel   convolution per channel, bias, activation, carried inputs; prompt portions and decode rows
//   rglru_kernel        bf16 on the tensor cores: gates of 128 channels and 64 tokens as one product, recurrence
//                       and GELU gate in the same kernel. A CTA keeps the gate weights of its channels in shared
//                       memory and walks a slice of the rows; where a portion runs over several slices, a first
//                       pass of the same kernel (kSummary) reduces each slice to its decay and end state
//   rglru_gates_any_kernel, rglru_scan_any_kernel   any sizes, fp32 or bf16 storage
//
// Channels: ``blocks`` parts of B (padded to a multiple of 16 with zeros: weights, hence channels and state).
#include "api.h"
#include "sm100.cuh"

namespace b200 {

typedef __nv_bfloat16 bf16;

template <typename T> struct Rg4;
template <> struct Rg4<float> {
  static __device__ __forceinline__ float4 get(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void put(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Rg4<bf16> {
  static __device__ __forceinline__ float4 get(const bf16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
  }
  static __device__ __forceinline__ void put(bf16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  }
};
__device__ __forceinline__ float rg_f(float v) { return v; }
__device__ __forceinline__ float rg_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void rg_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void rg_put(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float4 rg_fma(float4 a, float4 b, float4 c) {
  return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}

// -------------------------------------------------------------------------------- short convolution
static constexpr int kConvRun = 16;      // rows of a portion that one warp walks

// blockIdx.x: a decode row or a run of kConvRun rows of a portion; a warp takes 128 channels. The warp of a
// portion's first run also writes the new carried inputs, after its own reads of the old ones; later runs never
// look back past the portion's start (taps - 1 <= kConvRun).
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) short_conv_kernel(B200ShortConv p) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, c = (blockIdx.y * 4 + (threadIdx.x >> 5)) * 128 + lane * 4;
  const int taps = TAPS ? TAPS : p.taps;
  const B200Rows& R = p.rows;
  int req, row0, n, at, len;             // first row, rows, their offset in the portion, the portion's length
  if ((int)blockIdx.x < R.nd) {
    req = row0 = blockIdx.x;
    n = len = 1;
    at = 0;
  } else {
    const int u = blockIdx.x - R.nd, tile = u / (128 / kConvRun);
    const int r = R.tile_req[tile], b = R.q_start[r];
    at = R.tile_q0[tile] + (u % (128 / kConvRun)) * kConvRun;
    len = R.q_start[r + 1] - b;
    if (at >= len) return;
    req = R.nd + r;
    row0 = R.nd + b + at;
    n = min(kConvRun, len - at);
  }
  if (c >= p.C) return;
  // (what does not depend on the slot is asked for ahead of it)
  const int slot = R.slots[req];
  const bool init = R.seq_lens[req] > len;
  const T* x = reinterpret_cast<const T*>(p.x) + (size_t)(row0 - at) * p.ldx + c;      // the portion's first row
  const float* w = p.w + c;
  float4 hist[TAPS > 1 ? TAPS - 1 : 1], wt[TAPS ? TAPS : 1];
  if (TAPS) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wt[j] = *reinterpret_cast<const float4*>(w + (size_t)j * p.C);
  }
  const float4 first = Rg4<T>::get(x + (size_t)at * p.ldx);
  T* out = reinterpret_cast<T*>(p.out) + (size_t)row0 * p.ldo + c;
  if (slot < 0) {                        // (a padding row: its values only have to be finite)
    for (int r = 0; r < n; ++r) Rg4<T>::put(out + (size_t)r * p.ldo, make_float4(0.f, 0.f, 0.f, 0.f));
    return;
  }
  T* st = reinterpret_cast<T*>(p.state) + (size_t)slot * (taps - 1) * p.C + c;
  auto input = [&](int pos) {            // input of the portion's row pos (before it: the carried ones)
    if (pos >= 0) return Rg4<T>::get(x + (size_t)pos * p.ldx);
    if (!init) return make_float4(0.f, 0.f, 0.f, 0.f);
    return Rg4<T>::get(st + (size_t)(taps - 1 + pos) * p.C);
  };
  const float4 bias = p.bias ? *reinterpret_cast<const float4*>(p.bias + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  if (TAPS) {
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j) hist[j] = input(at - (TAPS - 1) + j);
  }
  for (int r = 0; r < n; ++r) {
    float4 a = bias;
    if (TAPS) {
      const float4 xin = r == 0 ? first : input(at + r);
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j) a = rg_fma(wt[j], hist[j], a);
      a = rg_fma(wt[TAPS ? TAPS - 1 : 0], xin, a);
#pragma unroll
      for (int j = 0; j + 2 < TAPS; ++j) hist[j] = hist[j + 1];
      if (TAPS > 1) hist[TAPS > 1 ? TAPS - 2 : 0] = xin;
    } else {
      for (int j = 0; j < taps; ++j)
        a = rg_fma(*reinterpret_cast<const float4*>(w + (size_t)j * p.C), input(at + r - (taps - 1) + j), a);
    }
    if (p.act == 1)
      a = make_float4(a.x / (1.f + expf(-a.x)), a.y / (1.f + expf(-a.y)), a.z / (1.f + expf(-a.z)), a.w / (1.f + expf(-a.w)));
    Rg4<T>::put(out + (size_t)r * p.ldo, a);
  }
  if (at == 0)                           // (ascending: entry i takes an input of the portion or the old entry len + i)
    for (int i = 0; i < taps - 1; ++i) Rg4<T>::put(st + (size_t)i * p.C, input(len - (taps - 1) + i));
}

// ------------------------------------------------------------------------- recurrence, any sizes
// a = exp(rate r), b = sqrt(1 - a^2) i u for 64 tokens and 32 channels of one block.
template <typename T>
__global__ void __launch_bounds__(256) rglru_gates_any_kernel(B200Rglru p) {
  __shared__ float sa[16][68], sw[16][68];
  __shared__ float lg[64][65];
  pdl_wait();
  pdl_launch_dependents();
  const int blk = blockIdx.z, m0 = blockIdx.y * 64, c0 = blockIdx.x * 32, C = p.blocks * p.B;
  const T* u = reinterpret_cast<const T*>(p.u) + (size_t)blk * p.B;
  const T* w = reinterpret_cast<const T*>(p.gates) + (size_t)blk * 2 * p.M * p.B;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < p.B; k0 += 16) {
    for (int x = threadIdx.x; x < 64 * 16; x += 256) {
      const int r = x >> 4, k = x & 15, ch = c0 + (r & 31);
      sa[k][r] = m0 + r < p.rows.T ? rg_f(u[(size_t)(m0 + r) * p.ldu + k0 + k]) : 0.f;
      sw[k][r] = ch < p.B ? rg_f(w[((size_t)(r >> 5) * p.M + ch) * p.B + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(sa[k][ty * 4 + i], sw[k][tx * 4 + j], acc[i][j]);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) lg[ty * 4 + i][tx * 4 + j] = acc[i][j];
  __syncthreads();
  for (int x = threadIdx.x; x < 64 * 32; x += 256) {
    const int m = m0 + (x >> 5), ch = c0 + (x & 31);
    if (m >= p.rows.T || ch >= p.B) continue;
    const int c = blk * p.B + ch;
    const float r = 1.f / (1.f + expf(-(lg[x >> 5][x & 31] + p.gate_bias[c])));
    const float g = 1.f / (1.f + expf(-(lg[x >> 5][32 + (x & 31)] + p.gate_bias[C + c])));
    const float la = p.rate[c] * r;
    p.a[(size_t)m * C + c] = expf(la);
    p.b[(size_t)m * C + c] = sqrtf(-expm1f(2.f * la)) * g * rg_f(u[(size_t)m * p.ldu + ch]);
  }
}

__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// One thread per request and channel walks the request's rows.
template <typename T>
__global__ void __launch_bounds__(128) rglru_scan_any_kernel(B200Rglru p) {
  pdl_wait();
  pdl_launch_dependents();
  const B200Rows& R = p.rows;
  const int C = p.blocks * p.B, c = blockIdx.y * 128 + threadIdx.x, req = blockIdx.x;
  if (c >= C) return;
  int row0 = req, n = 1;
  if (req >= R.nd) {
    const int b = R.q_start[req - R.nd];
    row0 = R.nd + b;
    n = R.q_start[req - R.nd + 1] - b;
  }
  const int slot = R.slots[req];
  float s = slot >= 0 && R.seq_lens[req] > n ? p.state[(size_t)slot * C + c] : 0.f;
  for (int t = row0; t < row0 + n; ++t) {
    s = fmaf(p.a[(size_t)t * C + c], s, p.b[(size_t)t * C + c]);
    rg_put(reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo + c,
           s * gelu_tanh_f(rg_f(reinterpret_cast<const T*>(p.y)[(size_t)t * p.ldy + c])));
  }
  if (slot >= 0) p.state[(size_t)slot * C + c] = s;
}

// ------------------------------------------------------------------ recurrence on the tensor cores
// One CTA: 128 channels of a block (blockIdx.x) and one slice of the units (blockIdx.y). A unit is up to 64
// rows: decode rows, or rows of one portion (half of a 128-row tile). Gate logits come out transposed, channels
// as the 128 rows of the product and tokens as its 64 columns, so that a thread holds one channel and walks
// its tokens in registers. Warps 0-15: recurrence, lane quarter = channels, four parts of 16 tokens; every part
// reduces its tokens to (decay, end state), the parts exchange these, and each runs through once more from the
// state it starts with. Warp 16: TMA, warp 17: MMA; the product of the next unit, its rows of y and the look-up of
// where its rows are run under the recurrence of this one.
static constexpr int kUnit = 64, kParts = 4, kPart = kUnit / kParts, kMaxUStages = 4;
static constexpr int kRgWarps = 4 * kParts, kRgThreads = (kRgWarps + 2) * 32;

struct alignas(8) RgBars {
  uint64_t w_full, u_full[kMaxUStages], u_empty[kMaxUStages], d_full[2], d_empty[2];
  uint32_t tmem_base;
  float2 xch[2][kParts][128];            // [unit parity][part][channel]: decay, end state
};

struct RgUnit {
  int row0, n, at, len, req;             // rows [row0, row0 + n); of a portion: their offset, its length
  bool decode;
};

__device__ __forceinline__ RgUnit rg_unit(const B200Rows& R, int i, int decode_units) {
  RgUnit u;
  u.decode = i < decode_units;
  if (u.decode) {
    u.row0 = i * kUnit;
    u.n = min(kUnit, R.nd - u.row0);
    u.at = u.len = u.req = 0;
    return u;
  }
  const int tile = (i - decode_units) >> 1, r = R.tile_req[tile], b = R.q_start[r];
  u.len = R.q_start[r + 1] - b;
  u.at = R.tile_q0[tile] + ((i - decode_units) & 1) * kUnit;
  u.n = max(0, min(kUnit, u.len - u.at));
  u.row0 = R.nd + b + u.at;
  u.req = R.nd + r;
  return u;
}

static constexpr float kRgLog2e = 1.4426950408889634f;

__device__ __forceinline__ float rg_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rg_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rg_sqrt(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// 1 - exp(x) for x <= 0, ex = exp(x): near 0 the series of expm1
__device__ __forceinline__ float rg_one_minus_exp(float x, float ex) {
  const float series = -x * fmaf(x, fmaf(x, fmaf(x, 1.f / 24.f, 1.f / 6.f), 0.5f), 1.f);
  return x > -0.02f ? series : 1.f - ex;
}
// w (1 + tanh z) / 2 with z = sqrt(2 / pi) (w + 0.044715 w^3), as w / (1 + exp(-2 z))
__device__ __forceinline__ float rg_gelu(float w) {
  const float k = -2.f * 0.7978845608028654f * kRgLog2e;
  return w * rg_rcp(1.f + rg_ex2(w * fmaf(w * w, 0.044715f * k, k)));
}
template <bool B> struct RgFlag { static constexpr bool value = B; };

template <bool kSummary>
__global__ void __launch_bounds__(kRgThreads, 1)
    rglru_kernel(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ CUtensorMap tmU, B200Rglru p, int units,
                 int per_slice, int stages, int* status) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int kc = (p.B + 63) / 64, ksteps = p.B / 16;
  uint8_t* sW = smem;                                   // [gate][chunk][128 rows x 64]
  uint8_t* sU = sW + 2 * kc * 16384;                    // [stage][chunk][64 rows x 64]
  RgBars* bars = reinterpret_cast<RgBars*>(sU + stages * kc * 8192);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int groups = p.M / 128, blk = blockIdx.x / groups, part = blockIdx.x % groups;
  const B200Rows& R = p.rows;
  const int decode_units = (R.nd + kUnit - 1) / kUnit, slice = blockIdx.y;
  const int unit0 = slice * per_slice, unit1 = min(units, unit0 + per_slice);
  const int C = p.blocks * p.B;

  if (threadIdx.x == 0) {
    mbar_init(&bars->w_full, 1);
    for (int i = 0; i < stages; ++i) { mbar_init(&bars->u_full[i], 1); mbar_init(&bars->u_empty[i], kRgWarps); }
    for (int i = 0; i < 2; ++i) { mbar_init(&bars->d_full[i], 1); mbar_init(&bars->d_empty[i], kRgWarps); }
    mbar_fence_init();
  }
  if (warp == kRgWarps + 1) { tmem_alloc(&bars->tmem_base, 256); tmem_relinquish(); }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = bars->tmem_base;                // buffer b: r logits at 128 b, i logits at 128 b + 64
  if (warp == kRgWarps && lane == 0) {                  // (weights: written by no kernel of the step)
    tma_prefetch_desc(&tmW);
    tma_prefetch_desc(&tmU);
    mbar_expect_tx(&bars->w_full, 2 * kc * 16384);
    for (int g = 0; g < 2; ++g)
      for (int c = 0; c < kc; ++c)
        tma_load_2d(sW + (g * kc + c) * 16384, &tmW, &bars->w_full, c * 64, (blk * 2 + g) * p.M + part * 128);
  }
  pdl_wait();
  pdl_launch_dependents();
  int first = unit0, last = unit1;
  if (kSummary) {
    // only a slice whose last portion runs on into the next slice, from that portion's start
    bool runs_on = false;
    int i = unit1 - 1;
    for (; i >= unit0; --i) {
      const RgUnit u = rg_unit(R, i, decode_units);
      if (u.decode) break;
      if (u.n > 0) { runs_on = u.at + u.n < u.len; first = max(unit0, i - u.at / kUnit); break; }
    }
    if (!runs_on || unit1 >= units) last = first;
  }

  if (warp == kRgWarps) {
    if (lane == 0) {
      int k = 0;
      for (int i = first; i < last; ++i) {
        const RgUnit u = rg_unit(R, i, decode_units);
        if (u.n <= 0) continue;
        const int st = k % stages;
        if (!mbar_wait(&bars->u_empty[st], ((k / stages) & 1) ^ 1, status)) break;
        mbar_expect_tx(&bars->u_full[st], kc * 8192);
        for (int c = 0; c < kc; ++c)
          tma_load_2d(sU + (st * kc + c) * 8192, &tmU, &bars->u_full[st], blk * p.B + c * 64, u.row0);
        ++k;
      }
      // (the weights must not be on their way when the block ends)
      if (k == 0) mbar_wait(&bars->w_full, 0, status);
    }
  } else if (warp == kRgWarps + 1) {
    if (lane == 0 && first < last) {
      const uint32_t idesc = umma_idesc_bf16(128, kUnit, 0, 0);
      const uint64_t wd0 = umma_desc_k_sw128(smem_u32(sW), 1024), ud0 = umma_desc_k_sw128(smem_u32(sU), 1024);
      bool ok = mbar_wait(&bars->w_full, 0, status);
      int k = 0;
      for (int i = first; i < last && ok; ++i) {
        const RgUnit u = rg_unit(R, i, decode_units);
        if (u.n <= 0) continue;
        const int st = k % stages, buf = k & 1;
        ok = mbar_wait(&bars->u_full[st], (k / stages) & 1, status) && mbar_wait(&bars->d_empty[buf], ((k >> 1) & 1) ^ 1, status);
        if (!ok) break;
        tc_fence_after_sync();
        const uint64_t ud = ud0 + ((st * kc * 8192) >> 4);
        for (int g = 0; g < 2; ++g)
          for (int s = 0; s < ksteps; ++s)
            umma_bf16_ss(tmem + buf * 128 + g * 64, wd0 + (((g * kc + (s >> 2)) * 16384) >> 4) + (s & 3) * 2,
                         ud + (((s >> 2) * 8192) >> 4) + (s & 3) * 2, idesc, s != 0);
        umma_commit(&bars->d_full[buf]);
        ++k;
      }
    }
  } else {
    const int quarter = warp & 3, piece = warp >> 2, ch = quarter * 32 + lane;      // channel of the tile
    const int cb = part * 128 + ch, c = blk * p.B + cb;                             // of the block, of all
    const bool live = cb < p.B;
    const uint32_t lane_off = (uint32_t)(quarter * 32) << 16;
    // (sigmoid(x + bias) as 1 / (1 + 2^(-log2(e) (x + bias))))
    const float bias_r = live ? -kRgLog2e * p.gate_bias[c] : 0.f, bias_i = live ? -kRgLog2e * p.gate_bias[C + c] : 0.f;
    const float rate = live ? p.rate[c] : 0.f, rate_l2 = rate * kRgLog2e;
    float* sum = p.summary + c;
    const size_t kind = (size_t)B200_RGLRU_SLICES * C;      // summary: end states | decays | starting states
    const bf16* y = reinterpret_cast<const bf16*>(p.y);
    bf16* out = reinterpret_cast<bf16*>(p.out);
    const uint32_t ldy = (uint32_t)p.ldy, ldo = (uint32_t)p.ldo;                    // (offsets below 2^31: checked)
    const int uc = min(cb >> 6, kc - 1), ux = (cb & 63) >> 3, uo = (cb & 7) * 2;    // u of this channel in a stage
    const int t0 = piece * kPart;
    float carry = 0.f, decay = 1.f;                         // state before the unit; kSummary: decay since the slice's start
    bool ok = true;
    int k = 0;
    bf16 yv[kPart];
    auto load_y = [&](const RgUnit& u) {
      const uint32_t at = (uint32_t)(u.row0 + t0) * ldy + c;
      if (live && t0 + kPart <= u.n) {
#pragma unroll
        for (int t = 0; t < kPart; ++t) yv[t] = y[at + t * ldy];
      } else {
#pragma unroll
        for (int t = 0; t < kPart; ++t) yv[t] = live && t0 + t < u.n ? y[at + t * ldy] : __float2bfloat16(0.f);
      }
    };
    RgUnit next = {};
    if (first < last) {
      next = rg_unit(R, first, decode_units);
      if (!kSummary) load_y(next);
    }
    for (int i = first; i < last; ++i) {
      const RgUnit u = next;
      if (i + 1 < last) next = rg_unit(R, i + 1, decode_units);
      if (u.n <= 0) {
        if (!kSummary && i + 1 < last) load_y(next);
        continue;
      }
      const int st = k % stages, buf = k & 1, n = min(max(u.n - t0, 0), kPart);
      float before[kPart];                                  // decode: the rows' states
      int slot = -1;                                        // decode: that of row t0 + lane
      if (!kSummary && u.decode) {
        bool fresh = true;
        if (lane < n) {
          slot = R.slots[u.row0 + t0 + lane];
          fresh = R.seq_lens[u.row0 + t0 + lane] <= 1;
        }
        const int from = fresh ? -1 : slot;
#pragma unroll
        for (int t = 0; t < kPart; ++t) {
          const int s = __shfl_sync(0xffffffffu, from, t);
          before[t] = live && s >= 0 ? p.state[(size_t)s * C + c] : 0.f;
        }
      } else if (u.at == 0) {                               // a portion starts
        const int s = R.slots[u.req];
        carry = 0.f;
        if (live && s >= 0 && R.seq_lens[u.req] > u.len) {
          // (a later slice may already have written the state of a portion that runs on: the first pass kept it)
          const bool runs_on = (i + (u.len + kUnit - 1) / kUnit) > unit1;
          carry = !kSummary && runs_on ? sum[2 * kind + (size_t)slice * C] : p.state[(size_t)s * C + c];
        }
        if (kSummary) {
          decay = 0.f;
          if (live && piece == 0) sum[2 * kind + (size_t)slice * C] = carry;
        }
      } else if (i == first && !kSummary && live) {         // a portion of earlier slices goes on
        const int from = (i - u.at / kUnit) / per_slice;
        carry = 0.f;
        for (int s = from; s < slice; ++s) carry = fmaf(sum[kind + (size_t)s * C], carry, sum[(size_t)s * C]);
      }
      ok = ok && __all_sync(0xffffffffu, mbar_wait(&bars->d_full[buf], (k >> 1) & 1, status));
      tc_fence_after_sync();
      uint32_t lr[kPart], li[kPart];
      tmem_ld_32x32b_x16(tmem + buf * 128 + t0 + lane_off, lr);
      tmem_ld_32x32b_x16(tmem + buf * 128 + 64 + t0 + lane_off, li);
      tmem_ld_wait();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->d_empty[buf]);
      const uint8_t* us = sU + (st * kc + uc) * 8192 + t0 * 128 + uo;
      float D = 1.f, S = 0.f;
      auto reduce = [&](auto full) {                        // decays to lr, inputs to li
#pragma unroll
        for (int t = 0; t < kPart; ++t) {
          const float r = rg_rcp(1.f + rg_ex2(fmaf(__uint_as_float(lr[t]), -kRgLog2e, bias_r)));
          const float g = rg_rcp(1.f + rg_ex2(fmaf(__uint_as_float(li[t]), -kRgLog2e, bias_i)));
          const float x = __bfloat162float(*reinterpret_cast<const bf16*>(us + t * 128 + ((ux ^ (t & 7)) << 4)));
          float a = rg_ex2(rate_l2 * r), b = rg_sqrt(rg_one_minus_exp(2.f * rate * r, a * a)) * (g * x);
          if (!decltype(full)::value && t >= n) { a = 1.f; b = 0.f; }
          lr[t] = __float_as_uint(a);
          li[t] = __float_as_uint(b);
          D *= a;
          S = fmaf(a, S, b);
        }
      };
      if (n == kPart) reduce(RgFlag<true>());
      else reduce(RgFlag<false>());
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->u_empty[st]);
      const uint32_t at = (uint32_t)(u.row0 + t0) * ldo + c;
      if (!kSummary && u.decode) {
#pragma unroll
        for (int t = 0; t < kPart; ++t) {
          const int to = __shfl_sync(0xffffffffu, slot, t);
          if (live && t < n) {
            const float s = fmaf(__uint_as_float(lr[t]), before[t], __uint_as_float(li[t]));
            out[at + t * ldo] = __float2bfloat16(s * rg_gelu(__bfloat162float(yv[t])));
            if (to >= 0) p.state[(size_t)to * C + c] = s;
          }
        }
      } else {
        bars->xch[k & 1][piece][ch] = make_float2(D, S);
        asm volatile("bar.sync 1, %0;" ::"n"(kRgWarps * 32) : "memory");
        float s = carry, end = carry;
#pragma unroll
        for (int q = 0; q < kParts; ++q) {
          const float2 h = bars->xch[k & 1][q][ch];
          if (q == piece) s = end;
          end = fmaf(h.x, end, h.y);
          if (kSummary) decay *= h.x;
        }
        if (!kSummary) {
          if (live && n == kPart) {
#pragma unroll
            for (int t = 0; t < kPart; ++t) {
              s = fmaf(__uint_as_float(lr[t]), s, __uint_as_float(li[t]));
              out[at + t * ldo] = __float2bfloat16(s * rg_gelu(__bfloat162float(yv[t])));
            }
          } else if (live) {
#pragma unroll
            for (int t = 0; t < kPart; ++t) {
              s = fmaf(__uint_as_float(lr[t]), s, __uint_as_float(li[t]));
              if (t < n) out[at + t * ldo] = __float2bfloat16(s * rg_gelu(__bfloat162float(yv[t])));
            }
          }
          if (live && piece == 0 && u.at + u.n >= u.len) {
            const int to = R.slots[u.req];
            if (to >= 0) p.state[(size_t)to * C + c] = end;
          }
        }
        carry = end;
      }
      if (!kSummary && i + 1 < last) load_y(next);          // (used at the end of the next unit)
      ++k;
    }
    if (kSummary && live && piece == 0 && first < last) {
      sum[(size_t)slice * C] = carry;
      sum[kind + (size_t)slice * C] = decay;
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  if (warp == kRgWarps + 1) tmem_dealloc(tmem, 256);
}

static size_t rg_smem(int B, int stages) {
  const int kc = (B + 63) / 64;
  return (size_t)2 * kc * 16384 + (size_t)stages * kc * 8192 + sizeof(RgBars) + 1024;
}
static int rg_units(const B200Rglru* a) { return (a->rows.nd + kUnit - 1) / kUnit + 2 * a->rows.num_tiles; }

}  // namespace b200

using namespace b200;

extern "C" {

int b200_short_conv(const B200ShortConv* a, cudaStream_t stream) {
  if (a->rows.T <= 0) return 0;
  if (a->C <= 0 || (a->C & 3) || (a->ldx & 3) || (a->ldo & 3) || a->taps < 1 || a->act < 0 || a->act > 1) return -1;
  if (a->taps - 1 > kConvRun) return -4;
  const dim3 grid(a->rows.nd + a->rows.num_tiles * (128 / kConvRun), (a->C + 511) / 512);
  if (grid.x == 0) return 0;
  auto go = [&](auto kernel) { return launch_pdl(kernel, grid, dim3(128), 0, stream, *a) == cudaSuccess ? 0 : -2; };
  if (a->f32) return a->taps == 4 ? go(short_conv_kernel<float, 4>) : go(short_conv_kernel<float, 0>);
  switch (a->taps) {
    case 2: return go(short_conv_kernel<bf16, 2>);
    case 3: return go(short_conv_kernel<bf16, 3>);
    case 4: return go(short_conv_kernel<bf16, 4>);
    default: return go(short_conv_kernel<bf16, 0>);
  }
}

// 1: the tensor-core kernel serves this shape.
int b200_rglru_fits(const B200Rglru* a) {
  return !a->f32 && a->B > 0 && a->B <= 256 && !(a->B & 15) && a->M % 128 == 0 && a->M >= a->B && !(a->ldu & 7) &&
         a->rows.T * a->ldy < (1ll << 31) && a->rows.T * a->ldo < (1ll << 31) && !(((uintptr_t)a->u | (uintptr_t)a->gates) & 15) && a->summary;
}

// Slices of the rows: one wave of CTAs over all channels.
int b200_rglru_slices(const B200Rglru* a) {
  const int groups = a->blocks * (a->M / 128), units = rg_units(a);
  int s = b200_num_sms() / (groups > 0 ? groups : 1);
  if (s > B200_RGLRU_SLICES) s = B200_RGLRU_SLICES;
  if (s > units) s = units;
  return s < 1 ? 1 : s;
}

int b200_rglru(const B200Rglru* a, int any_size, cudaStream_t stream) {
  if (a->rows.T <= 0) return 0;
  const int C = a->blocks * a->B;
  if (a->blocks <= 0 || a->B <= 0 || (a->B & 15) || a->M < a->B || a->ldu < C || a->ldo < C || a->ldy < C) return -1;
  if (any_size || !b200_rglru_fits(a)) {
    if (!a->a || !a->b) return -1;
    const dim3 g1((a->B + 31) / 32, (a->rows.T + 63) / 64, a->blocks);
    const dim3 g2(a->rows.nd + a->rows.num_prefills, (C + 127) / 128);
    if (g1.y > 65535 || g1.z > 65535 || g2.y > 65535) return -4;
    if (g2.x == 0) return 0;
    auto go = [&](auto gates, auto scan) {
      if (launch_pdl(gates, g1, dim3(256), 0, stream, *a) != cudaSuccess) return -2;
      return launch_pdl(scan, g2, dim3(128), 0, stream, *a) == cudaSuccess ? 0 : -2;
    };
    return a->f32 ? go(rglru_gates_any_kernel<float>, rglru_scan_any_kernel<float>)
                  : go(rglru_gates_any_kernel<bf16>, rglru_scan_any_kernel<bf16>);
  }
  const int units = rg_units(a);
  if (units == 0) return 0;
  CUtensorMap tmW, tmU;
  if (!encode_tmap_2d(&tmW, a->gates, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (uint64_t)a->blocks * 2 * a->M, a->B, a->B, 128, 64,
                      CU_TENSOR_MAP_SWIZZLE_128B) ||
      !encode_tmap_2d(&tmU, a->u, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (uint64_t)a->rows.T, C, (uint64_t)a->ldu, kUnit, 64,
                      CU_TENSOR_MAP_SWIZZLE_128B))
    return -3;
  const int groups = a->blocks * (a->M / 128);
  int slices = b200_rglru_slices(a);
  const int per = (units + slices - 1) / slices;
  slices = (units + per - 1) / per;
  int stages = kMaxUStages;
  while (stages > 2 && rg_smem(a->B, stages) > 227 * 1024) --stages;
  const size_t smem = rg_smem(a->B, stages);
  static PerDeviceOnce once;
  if (once.first()) {
    cudaFuncSetAttribute(rglru_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    cudaFuncSetAttribute(rglru_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
  }
  const dim3 grid(groups, slices);
  int* st = device_status_word();
  if (slices > 1 && a->rows.num_tiles > 0 &&
      launch_pdl(rglru_kernel<true>, grid, dim3(kRgThreads), smem, stream, tmW, tmU, *a, units, per, stages, st) != cudaSuccess)
    return -2;
  return launch_pdl(rglru_kernel<false>, grid, dim3(kRgThreads), smem, stream, tmW, tmU, *a, units, per, stages, st) ==
                 cudaSuccess ? 0 : -2;
}

}  // extern "C"
