// Gated delta rule with per-layer sizes, everything that enters the recurrence in fp32.
//
//   delta_prep_kernel   short causal convolutions (any number of taps) + SiLU, unit q / k per head, log
//                       decay and write strength, convolution state; prompt portions and decode rows
//   delta_rule_kernel   with F = e^g S the faded state:  S = F + k (x) beta (v - k F),  o = q S  token by token,
//                       the state in registers, then RMS norm of o, weight and SiLU gate. Serves decode rows
//                       and, for any sizes and fp32 storage, whole prompt portions
//   delta_norm_kernel   the same norm and gate over rows of fp32 o (after the chunked prompt kernel)
//
// Sizes D, V are padded to multiples of 16 with zeros (weights, hence activations and state); ``dim`` and
// ``vdim`` are the sizes the norms divide by. Rows: the first nd rows are decode rows (one per request), then
// the prompt portions in request order. State [slots][H][D][V] fp32, convolution state [slots][taps - 1][C].
#include "api.h"
#include "sm100.cuh"

namespace b200 {

typedef __nv_bfloat16 bf16;

static constexpr int kRun = 16;        // rows of a portion that one warp of the preparation walks
static constexpr int kMaxChannels = 512;

template <typename T> struct Ld4;
template <> struct Ld4<float> {
  static __device__ __forceinline__ float4 get(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void put(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Ld4<bf16> {
  static __device__ __forceinline__ float4 get(const bf16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
  }
  static __device__ __forceinline__ void put(bf16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  }
};
__device__ __forceinline__ float4 fma4(float4 a, float4 b, float4 c) {
  return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}
__device__ __forceinline__ float4 fma4(float a, float4 b, float4 c) { return fma4(make_float4(a, a, a, a), b, c); }
__device__ __forceinline__ float4 mul4(float a, float4 b) { return make_float4(a * b.x, a * b.y, a * b.z, a * b.w); }
__device__ __forceinline__ float sq4(float4 a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }
__device__ __forceinline__ float silu1(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float4 silu4(float4 a) { return make_float4(silu1(a.x), silu1(a.y), silu1(a.z), silu1(a.w)); }
__device__ __forceinline__ float softplus1(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// ------------------------------------------------------------------------------------ preparation
// blockIdx.x: a decode row or a run of kRun rows of a portion; a warp takes one section of channels (a q, k
// or v head) or the gates. The warp of a portion's first run also writes the new convolution state, after
// its own reads of the old one; later runs never look back past the portion's start (taps - 1 <= kRun).
template <typename T, int NI, int TAPS>
__global__ void __launch_bounds__(128) delta_prep_kernel(B200Delta p) {
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sec = blockIdx.y * 4 + warp;
  const int nsec = 2 * p.G + p.H, taps = TAPS ? TAPS : p.taps;
  if (sec > nsec) return;
  int req, row0, n, at, len;            // first row, rows, their offset in the portion, the portion's length
  if ((int)blockIdx.x < p.nd) {
    req = row0 = blockIdx.x;
    n = len = 1;
    at = 0;
  } else {
    const int u = blockIdx.x - p.nd, tile = u / (128 / kRun);
    const int r = p.tile_req[tile], b = p.q_start[r];
    at = p.tile_q0[tile] + (u % (128 / kRun)) * kRun;
    len = p.q_start[r + 1] - b;
    if (at >= len) return;
    req = p.nd + r;
    row0 = p.nd + b + at;
    n = min(kRun, len - at);
  }
  const int slot = p.slots[req];
  if (slot < 0) return;
  const bool init = p.seq_lens[req] > len;
  if (sec == nsec) {
    for (int i = lane; i < n * p.H; i += 32) {
      const int t = row0 + i / p.H, h = i % p.H;
      const float* ab = p.ab + (size_t)t * p.ldab;
      p.g[(size_t)t * p.H + h] = -p.A[h] * softplus1(ab[h] + p.dt[h]);
      p.beta[(size_t)t * p.H + h] = 1.f / (1.f + expf(-ab[p.H + h]));
    }
    return;
  }
  const bool is_v = sec >= 2 * p.G;
  const int width = is_v ? p.V : p.D, c0 = is_v ? 2 * p.G * p.D + (sec - 2 * p.G) * p.V : sec * p.D;
  const int C = 2 * p.G * p.D + p.H * p.V;
  const T* x = reinterpret_cast<const T*>(p.proj) + (size_t)(row0 - at) * p.ldp + c0;   // the portion's first row
  T* st = reinterpret_cast<T*>(p.conv_state) + (size_t)slot * (taps - 1) * C + c0;
  const float* w = p.conv_w + c0;
  auto input = [&](int pos, int c) {     // input of the portion's row pos (before it: the state)
    if (pos >= 0) return Ld4<T>::get(x + (size_t)pos * p.ldp + c);
    if (!init) return make_float4(0.f, 0.f, 0.f, 0.f);
    return Ld4<T>::get(st + (size_t)(taps - 1 + pos) * C + c);
  };
  float4 hist[TAPS > 1 ? TAPS - 1 : 1][NI], wt[TAPS ? TAPS : 1][NI];
  if (TAPS) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = i * 128 + lane * 4;
      if (c < width) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) wt[j][i] = *reinterpret_cast<const float4*>(w + (size_t)j * C + c);
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) hist[j][i] = input(at - (TAPS - 1) + j, c);
      }
    }
  }
  for (int r = 0; r < n; ++r) {
    float4 y[NI];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = i * 128 + lane * 4;
      if (c >= width) continue;
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      if (TAPS) {
        const float4 xin = input(at + r, c);
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) a = fma4(wt[j][i], hist[j][i], a);
        a = fma4(wt[TAPS ? TAPS - 1 : 0][i], xin, a);
#pragma unroll
        for (int j = 0; j + 2 < TAPS; ++j) hist[j][i] = hist[j + 1][i];
        if (TAPS > 1) hist[TAPS > 1 ? TAPS - 2 : 0][i] = xin;
      } else {
        for (int j = 0; j < taps; ++j)
          a = fma4(*reinterpret_cast<const float4*>(w + (size_t)j * C + c), input(at + r - (taps - 1) + j, c), a);
      }
      y[i] = silu4(a);
      ss += sq4(y[i]);
    }
    const size_t t = row0 + r;
    if (is_v) {
      T* d = reinterpret_cast<T*>(p.v) + (t * p.H + sec - 2 * p.G) * p.V;
#pragma unroll
      for (int i = 0; i < NI; ++i)
        if (i * 128 + lane * 4 < width) Ld4<T>::put(d + i * 128 + lane * 4, y[i]);
    } else {
      float inv = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
      if (sec < p.G) inv *= p.q_scale;
      float* d = (sec < p.G ? p.q + (t * p.G + sec) * p.D : p.k + (t * p.G + sec - p.G) * p.D);
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int c = i * 128 + lane * 4;
        if (c >= width) continue;
        const float4 x = mul4(inv, y[i]);
        if (p.split && (int)blockIdx.x >= p.nd) {        // x = hi + lo
          bf16* b = reinterpret_cast<bf16*>(d) + c;
          Ld4<bf16>::put(b, x);
          const float4 hi = Ld4<bf16>::get(b);
          Ld4<bf16>::put(b + p.D, make_float4(x.x - hi.x, x.y - hi.y, x.z - hi.z, x.w - hi.w));
        } else {
          *reinterpret_cast<float4*>(d + c) = x;
        }
      }
    }
  }
  if (at == 0) {
    // (ascending: entry i takes an input of the portion or the old entry len + i)
    for (int i = 0; i < taps - 1; ++i)
#pragma unroll
      for (int x4 = 0; x4 < NI; ++x4) {
        const int c = x4 * 128 + lane * 4;
        if (c < width) Ld4<T>::put(st + (size_t)i * C + c, input(len - (taps - 1) + i, c));
      }
  }
}

// -------------------------------------------------------------------------------- token by token
// Norm, weight and gate of one head's o, held in shared memory: written as T.
template <typename T>
__device__ __forceinline__ void gated_norm(const B200Delta& p, const float* o, float ss, size_t t, int h, int tid, int nt) {
  const float inv = 1.f / sqrtf(ss / (float)p.vdim + p.eps);
  const T* z = reinterpret_cast<const T*>(p.gate) + t * p.ldp + (size_t)h * p.V;
  T* out = reinterpret_cast<T*>(p.out) + t * p.ldo + (size_t)h * p.V;
  for (int c = tid * 4; c < p.V; c += nt * 4) {
    const float4 w = *reinterpret_cast<const float4*>(p.norm_w + c), g = silu4(Ld4<T>::get(z + c));
    const float4 x = *reinterpret_cast<const float4*>(o + c);
    Ld4<T>::put(out + c, make_float4(x.x * inv * w.x * g.x, x.y * inv * w.y * g.y, x.z * inv * w.z * g.z, x.w * inv * w.w * g.w));
  }
}

// grid (requests, H). Thread (v4, slice) holds rows [slice * rps, ...) of four state columns: in registers
// (MAXR rows) or, for states that do not fit, in memory.
template <typename T, int MAXR, int THREADS>
__global__ void __launch_bounds__(THREADS) delta_rule_kernel(B200Delta p, int slices, int rps) {
  extern __shared__ float4 rule_smem[];
  const int nv = p.V / 4;
  float* sk = reinterpret_cast<float*>(rule_smem);                 // [D]
  float* sq = sk + p.D;                                            // [D]
  float* so = sq + p.D;                                            // [V]
  float4* red0 = reinterpret_cast<float4*>(so + p.V);              // [slices][nv]
  float4* red1 = red0 + slices * nv;
  __shared__ float wsum[THREADS / 32];
  pdl_wait();
  pdl_launch_dependents();
  const int tid = threadIdx.x, h = blockIdx.y, kv = h / (p.H / p.G), v4 = tid % nv, sl = tid / nv;
  int req = blockIdx.x, t0 = req, len = 1;
  if (req >= p.nd) {
    t0 = p.nd + p.q_start[req - p.nd];
    len = p.q_start[req - p.nd + 1] - p.q_start[req - p.nd];
  }
  const int slot = p.slots[req];
  if (slot < 0) {                        // a padding row
    for (int t = t0; t < t0 + len; ++t)
      for (int c = tid; c < p.V; c += THREADS)
        reinterpret_cast<T*>(p.out)[(size_t)t * p.ldo + (size_t)h * p.V + c] = T(0.f);
    return;
  }
  const bool init = p.seq_lens[req] > len, on = sl < slices;
  const int r0 = sl * rps, nr = on ? max(0, min(rps, p.D - r0)) : 0;
  float4* S = reinterpret_cast<float4*>(p.state + ((size_t)slot * p.H + h) * p.D * p.V) + (size_t)r0 * nv + v4;
  float4 s[MAXR ? MAXR : 1];
  if (MAXR) {
#pragma unroll
    for (int r = 0; r < MAXR; ++r) s[r] = init && r < nr ? S[(size_t)r * nv] : make_float4(0.f, 0.f, 0.f, 0.f);
  } else if (!init) {
    for (int r = 0; r < nr; ++r) S[(size_t)r * nv] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int t = t0; t < t0 + len; ++t) {
    for (int i = tid; i < p.D; i += THREADS) {
      sk[i] = p.k[((size_t)t * p.G + kv) * p.D + i];
      sq[i] = p.q[((size_t)t * p.G + kv) * p.D + i];
    }
    const float lg = p.g[(size_t)t * p.H + h], beta = p.beta[(size_t)t * p.H + h];
    // A factor near one, applied over thousands of tokens, must not be rounded to fp32 first: its
    // distance from one is what is multiplied and added.
    const bool slow = lg > -0.5f;
    const float keep = slow ? 1.f : 0.f, rest = slow ? expm1f(lg) : expf(lg);
    auto decayed = [&](float4 x) { return fma4(rest, x, mul4(keep, x)); };
    __syncthreads();
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (MAXR) {
#pragma unroll
      for (int r = 0; r < MAXR; ++r)
        if (r < nr) {
          s[r] = decayed(s[r]);
          a = fma4(sk[r0 + r], s[r], a);
        }
    } else {
      for (int r = 0; r < nr; ++r) a = fma4(sk[r0 + r], decayed(S[(size_t)r * nv]), a);
    }
    if (on) red0[sl * nv + v4] = a;
    __syncthreads();
    if (on) {
      float4 u = Ld4<T>::get(reinterpret_cast<const T*>(p.v) + ((size_t)t * p.H + h) * p.V + v4 * 4);
      for (int x = 0; x < slices; ++x) {
        const float4 b = red0[x * nv + v4];
        u.x -= b.x; u.y -= b.y; u.z -= b.z; u.w -= b.w;
      }
      u = mul4(beta, u);
      a = make_float4(0.f, 0.f, 0.f, 0.f);
      if (MAXR) {
#pragma unroll
        for (int r = 0; r < MAXR; ++r)
          if (r < nr) {
            s[r] = fma4(sk[r0 + r], u, s[r]);
            a = fma4(sq[r0 + r], s[r], a);
          }
      } else {
        for (int r = 0; r < nr; ++r) {
          const float4 x = fma4(sk[r0 + r], u, decayed(S[(size_t)r * nv]));
          S[(size_t)r * nv] = x;
          a = fma4(sq[r0 + r], x, a);
        }
      }
      red1[sl * nv + v4] = a;
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < p.V; c += THREADS) {
      float o = 0.f;
      for (int x = 0; x < slices; ++x) o += reinterpret_cast<const float*>(red1)[x * p.V + c];
      so[c] = o;
      ss += o * o;
    }
    ss = warp_sum(ss);
    if ((tid & 31) == 0) wsum[tid >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int x = 0; x < THREADS / 32; ++x) ss += wsum[x];
    gated_norm<T>(p, so, ss, t, h, tid, THREADS);
  }
  if (MAXR) {
#pragma unroll
    for (int r = 0; r < MAXR; ++r)
      if (r < nr) S[(size_t)r * nv] = s[r];
  }
}

// One warp per (row, head) of fp32 o.
template <typename T>
__global__ void __launch_bounds__(128) delta_norm_kernel(B200Delta p, int rows) {
  pdl_wait();
  pdl_launch_dependents();
  const long x = (long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (x >= (long)rows * p.H) return;
  const size_t t = p.nd + x / p.H;
  const int h = (int)(x % p.H);
  const float* o = p.o + (t * p.H + h) * p.V;
  float ss = 0.f;
  for (int c = lane * 4; c < p.V; c += 128) ss += sq4(*reinterpret_cast<const float4*>(o + c));
  gated_norm<T>(p, o, warp_sum(ss), t, h, lane, 32);
}

static bool delta_ok(const B200Delta* a) {
  return a->G > 0 && a->H > 0 && a->H % a->G == 0 && a->D > 0 && a->V > 0 && !(a->D & 15) && !(a->V & 15) &&
         a->dim > 0 && a->vdim > 0 && a->dim <= a->D && a->vdim <= a->V && a->D <= kMaxChannels && a->V <= kMaxChannels &&
         a->taps >= 1 && a->taps <= kRun + 1 && !(a->ldp & 3) && !(a->ldo & 3);
}

template <typename T, int NI>
static cudaError_t launch_prep(const B200Delta& a, dim3 grid, cudaStream_t stream) {
  return a.taps == 4 ? launch_pdl(delta_prep_kernel<T, NI, 4>, grid, dim3(128), 0, stream, a)
                     : launch_pdl(delta_prep_kernel<T, NI, 0>, grid, dim3(128), 0, stream, a);
}
template <typename T>
static cudaError_t launch_prep(const B200Delta& a, dim3 grid, cudaStream_t stream) {
  const int w = a.D > a.V ? a.D : a.V;
  return w <= 128 ? launch_prep<T, 1>(a, grid, stream) : w <= 256 ? launch_prep<T, 2>(a, grid, stream)
                                                                  : launch_prep<T, 4>(a, grid, stream);
}
template <typename T>
static cudaError_t launch_rule(const B200Delta& a, int reqs, cudaStream_t stream) {
  const int nv = a.V / 4;
  // slices of the state's rows: at least 8 rows each
  int threads = 256;
  auto cut = [&](int& slices, int& rps) {
    slices = threads / nv;
    if (slices > (a.D + 7) / 8) slices = (a.D + 7) / 8;
    if (slices < 1) slices = 1;
    rps = (a.D + slices - 1) / slices;
  };
  int slices, rps;
  cut(slices, rps);
  if (rps > 32) { threads = 512; cut(slices, rps); }
  const size_t smem = (size_t)(2 * a.D + a.V + 2 * slices * a.V) * 4;
  const dim3 grid(reqs, a.H);
  if (threads == 512)
    return rps <= 32 ? launch_pdl(delta_rule_kernel<T, 32, 512>, grid, dim3(512), smem, stream, a, slices, rps)
                     : launch_pdl(delta_rule_kernel<T, 0, 512>, grid, dim3(512), smem, stream, a, slices, rps);
  if (rps <= 8) return launch_pdl(delta_rule_kernel<T, 8, 256>, grid, dim3(256), smem, stream, a, slices, rps);
  if (rps <= 16) return launch_pdl(delta_rule_kernel<T, 16, 256>, grid, dim3(256), smem, stream, a, slices, rps);
  return launch_pdl(delta_rule_kernel<T, 32, 256>, grid, dim3(256), smem, stream, a, slices, rps);
}

}  // namespace b200

using namespace b200;

extern "C" {

int b200_delta_prepare(const B200Delta* a, cudaStream_t stream) {
  const int units = a->nd + a->num_tiles * (128 / kRun);
  if (units <= 0) return 0;
  if (!delta_ok(a)) return -1;
  const dim3 grid(units, (2 * a->G + a->H + 1 + 3) / 4);
  return (a->f32 ? launch_prep<float>(*a, grid, stream) : launch_prep<bf16>(*a, grid, stream)) == cudaSuccess ? 0 : -2;
}

// reqs: the first of them that are run here (the decode rows, or those and the portions).
int b200_delta_rule(const B200Delta* a, int reqs, cudaStream_t stream) {
  if (reqs <= 0) return 0;
  if (!delta_ok(a)) return -1;
  return (a->f32 ? launch_rule<float>(*a, reqs, stream) : launch_rule<bf16>(*a, reqs, stream)) == cudaSuccess ? 0 : -2;
}

// rows: those after the decode rows.
int b200_delta_norm(const B200Delta* a, int rows, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (!delta_ok(a)) return -1;
  const dim3 grid((unsigned)(((long)rows * a->H + 3) / 4));
  return (a->f32 ? launch_pdl(delta_norm_kernel<float>, grid, dim3(128), 0, stream, *a, rows)
                 : launch_pdl(delta_norm_kernel<bf16>, grid, dim3(128), 0, stream, *a, rows)) == cudaSuccess ? 0 : -2;
}

}  // extern "C"
