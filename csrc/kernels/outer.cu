// Recurrences over outer products with fp32 states, S <- decay S + k v^T, o = S^T q (prompts in chunks: outer_chunk.cu).
//
//   outer_step_kernel   token by token, the state in registers: decode rows and, for any sizes and fp32 storage, whole
//                       prompt portions. Decay per key channel: with its low-rank product, output norm and gate. Decay per
//                       head: with the step size
//   outer_head_norm kernels  norm per head, weight and SiLU gate over rows of fp32 o
//   outer_part_norm_kernel   skip, SiLU gate, norm in equal parts over rows of fp32 o
//
// D and V are multiples of 16 padded with zeros; ``vdim`` is what the norms divide by.
#include "api.h"
#include "sm100.cuh"

namespace b200 {

typedef __nv_bfloat16 bf16;

template <typename T> struct Ou4;
template <> struct Ou4<float> {
  static __device__ __forceinline__ float4 get(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void put(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Ou4<bf16> {
  static __device__ __forceinline__ float4 get(const bf16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
  }
  static __device__ __forceinline__ void put(bf16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  }
};
__device__ __forceinline__ float ou_f(float v) { return v; }
__device__ __forceinline__ float ou_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float4 ou_fma(float4 a, float4 b, float4 c) {
  return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}
__device__ __forceinline__ float4 ou_fma(float a, float4 b, float4 c) { return ou_fma(make_float4(a, a, a, a), b, c); }
__device__ __forceinline__ float4 ou_mul(float a, float4 b) { return make_float4(a * b.x, a * b.y, a * b.z, a * b.w); }
__device__ __forceinline__ float ou_silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float4 ou_silu(float4 a) { return make_float4(ou_silu(a.x), ou_silu(a.y), ou_silu(a.z), ou_silu(a.w)); }
__device__ __forceinline__ float ou_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float ou_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Norm, weight and gate of one head's o.
template <typename T>
__device__ __forceinline__ void head_norm(const B200Outer& p, const float* o, float ss, size_t t, int h, int tid, int nt) {
  const float inv = 1.f / sqrtf(ss / (float)p.vdim + p.eps);
  const T* z = reinterpret_cast<const T*>(p.gate) + t * p.ldg + (size_t)h * p.V;
  T* out = reinterpret_cast<T*>(p.out) + t * p.ldo + (size_t)h * p.V;
  for (int c = tid * 4; c < p.V; c += nt * 4) {
    const float4 w = *reinterpret_cast<const float4*>(p.norm_w + c), g = ou_silu(Ou4<T>::get(z + c));
    const float4 x = *reinterpret_cast<const float4*>(o + c);
    Ou4<T>::put(out + c, make_float4(x.x * inv * w.x * g.x, x.y * inv * w.y * g.y, x.z * inv * w.z * g.z, x.w * inv * w.w * g.w));
  }
}

// -------------------------------------------------------------------------------- token by token
// grid (requests, H). Thread (v4, slice) holds rows [slice * rps, ...) of four state columns: in registers
// (MAXR rows) or, for states that do not fit, in memory.
template <typename T, int KIND, int MAXR, int THREADS>
__global__ void __launch_bounds__(THREADS) outer_step_kernel(B200Outer p, int slices, int rps) {
  extern __shared__ float4 step_smem[];
  const int nv = p.V / 4;
  float* sk = reinterpret_cast<float*>(step_smem);                 // [D]
  float* sq = sk + p.D;                                            // [D]
  float* s_rest = sq + p.D;                                        // [D] decay, or its distance from one (s_keep = 1)
  float* s_keep = s_rest + p.D;                                    // [D]
  float* so = s_keep + p.D;                                        // [V]
  float4* red = reinterpret_cast<float4*>(so + p.V);               // [slices][nv]
  __shared__ float wsum[THREADS / 32];
  pdl_wait();
  pdl_launch_dependents();
  const int tid = threadIdx.x, h = blockIdx.y, g = h / (p.H / p.G), v4 = tid % nv, sl = tid / nv;
  const B200Rows& R = p.rows;
  int req = blockIdx.x, t0 = req, len = 1;
  if (req >= R.nd) {
    t0 = R.nd + R.q_start[req - R.nd];
    len = R.q_start[req - R.nd + 1] - R.q_start[req - R.nd];
  }
  const int slot = R.slots[req];
  if (slot < 0) {                        // a padding row
    for (int t = t0; t < t0 + len; ++t)
      for (int c = tid; c < p.V; c += THREADS) {
        if (KIND == 0) reinterpret_cast<T*>(p.out)[(size_t)t * p.ldo + (size_t)h * p.V + c] = T(0.f);
        else p.o[((size_t)t * p.H + h) * p.V + c] = 0.f;
      }
    return;
  }
  const bool init = R.seq_lens[req] > len, on = sl < slices;
  const int r0 = sl * rps, nr = on ? max(0, min(rps, p.D - r0)) : 0;
  float4* S = reinterpret_cast<float4*>(p.state + ((size_t)slot * p.H + h) * p.D * p.V) + (size_t)r0 * nv + v4;
  float4 s[MAXR ? MAXR : 1];
  if (MAXR) {
#pragma unroll
    for (int r = 0; r < MAXR; ++r) s[r] = init && r < nr ? S[(size_t)r * nv] : make_float4(0.f, 0.f, 0.f, 0.f);
  } else if (!init) {
    for (int r = 0; r < nr; ++r) S[(size_t)r * nv] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const T* q = reinterpret_cast<const T*>(p.q) + (size_t)g * p.D;
  const T* k = reinterpret_cast<const T*>(p.k) + (size_t)g * p.D;
  const T* v = reinterpret_cast<const T*>(p.v) + (size_t)h * p.V;
  for (int t = t0; t < t0 + len; ++t) {
    // A factor near one, applied over thousands of tokens, must not be rounded to fp32 first: its distance from
    // one is what is multiplied and added.
    auto factor = [](float lg, float& keep, float& rest) {
      const bool slow = lg > -0.5f;
      keep = slow ? 1.f : 0.f;
      rest = slow ? expm1f(lg) : expf(lg);
    };
    float keep = 0.f, rest = 0.f, dt = 1.f;
    if (KIND == 1) {
      dt = ou_softplus(ou_f(reinterpret_cast<const T*>(p.dt)[(size_t)t * p.lddt + h]) + p.dt_bias[h]);
      factor(-p.A[h] * dt, keep, rest);
    }
    for (int i = tid; i < p.D; i += THREADS) {
      sk[i] = dt * ou_f(k[(size_t)t * p.ld + i]);
      sq[i] = p.q_scale * ou_f(q[(size_t)t * p.ld + i]);
      if (KIND == 0) {
        const T* a1 = reinterpret_cast<const T*>(p.a1) + (size_t)t * p.lda1;
        const T* a2 = reinterpret_cast<const T*>(p.a2) + ((size_t)h * p.D + i) * p.rank;
        float z = p.a2b[h * p.D + i];
        for (int r = 0; r < p.rank; r += 4) {
          const float4 x = Ou4<T>::get(a1 + r), w = Ou4<T>::get(a2 + r);
          z = fmaf(x.x, w.x, fmaf(x.y, w.y, fmaf(x.z, w.z, fmaf(x.w, w.w, z))));
        }
        factor(-ou_softplus(-z) * p.inv_tau, s_keep[i], s_rest[i]);
      }
    }
    const float4 vt = on ? Ou4<T>::get(v + (size_t)t * p.ld + v4 * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    __syncthreads();
    auto next = [&](float4 x, int r) {
      const float f = KIND == 0 ? s_rest[r0 + r] : rest, e = KIND == 0 ? s_keep[r0 + r] : keep;
      return ou_fma(sk[r0 + r], vt, ou_fma(f, x, ou_mul(e, x)));
    };
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (MAXR) {
#pragma unroll
      for (int r = 0; r < MAXR; ++r)
        if (r < nr) {
          s[r] = next(s[r], r);
          a = ou_fma(sq[r0 + r], s[r], a);
        }
    } else {
      for (int r = 0; r < nr; ++r) {
        const float4 x = next(S[(size_t)r * nv], r);
        S[(size_t)r * nv] = x;
        a = ou_fma(sq[r0 + r], x, a);
      }
    }
    if (on) red[sl * nv + v4] = a;
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < p.V; c += THREADS) {
      float o = 0.f;
      for (int x = 0; x < slices; ++x) o += reinterpret_cast<const float*>(red)[x * p.V + c];
      if (KIND == 1) p.o[((size_t)t * p.H + h) * p.V + c] = o;
      so[c] = o;
      ss = fmaf(o, o, ss);
    }
    if (KIND == 0) {
      ss = ou_sum(ss);
      if ((tid & 31) == 0) wsum[tid >> 5] = ss;
      __syncthreads();
      ss = 0.f;
#pragma unroll
      for (int x = 0; x < THREADS / 32; ++x) ss += wsum[x];
      head_norm<T>(p, so, ss, t, h, tid, THREADS);
    }
  }
  if (MAXR) {
#pragma unroll
    for (int r = 0; r < MAXR; ++r)
      if (r < nr) S[(size_t)r * nv] = s[r];
  }
}

// ------------------------------------------------------------------------------------------- norms
// Heads of up to 128 values: a warp takes kNormItems (row, head) pairs, loads first.
static constexpr int kNormItems = 4;
template <typename T>
__global__ void __launch_bounds__(128) outer_head_norm_vec_kernel(B200Outer p, int row0, uint32_t items) {
  pdl_wait();
  pdl_launch_dependents();
  const uint32_t x0 = (blockIdx.x * 4 + (threadIdx.x >> 5)) * kNormItems, H = p.H;
  const int c = (threadIdx.x & 31) * 4;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 o[kNormItems], z[kNormItems];
  const float4 w = c < p.V ? *reinterpret_cast<const float4*>(p.norm_w + c) : zero;
  T* to[kNormItems];
#pragma unroll
  for (int i = 0; i < kNormItems; ++i) {
    o[i] = z[i] = zero;
    to[i] = nullptr;
    if (x0 + i >= items || c >= p.V) continue;
    const uint32_t r = (x0 + i) / H, h = x0 + i - r * H;
    const size_t t = row0 + r;
    o[i] = *reinterpret_cast<const float4*>(p.o + (t * p.H + h) * p.V + c);
    z[i] = Ou4<T>::get(reinterpret_cast<const T*>(p.gate) + t * p.ldg + h * p.V + c);
    to[i] = reinterpret_cast<T*>(p.out) + t * p.ldo + h * p.V + c;
  }
#pragma unroll
  for (int i = 0; i < kNormItems; ++i) {
    const float ss = ou_sum(o[i].x * o[i].x + o[i].y * o[i].y + o[i].z * o[i].z + o[i].w * o[i].w);
    const float inv = 1.f / sqrtf(ss / (float)p.vdim + p.eps);
    const float4 g = ou_silu(z[i]);
    if (to[i])
      Ou4<T>::put(to[i], make_float4(o[i].x * inv * w.x * g.x, o[i].y * inv * w.y * g.y, o[i].z * inv * w.z * g.z, o[i].w * inv * w.w * g.w));
  }
}

// One warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(128) outer_head_norm_kernel(B200Outer p, int row0, int rows) {
  pdl_wait();
  pdl_launch_dependents();
  const long x = (long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (x >= (long)rows * p.H) return;
  const size_t t = row0 + x / p.H;
  const int h = (int)(x % p.H);
  const float* o = p.o + (t * p.H + h) * p.V;
  float ss = 0.f;
  for (int c = lane * 4; c < p.V; c += 128) {
    const float4 v = *reinterpret_cast<const float4*>(o + c);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  head_norm<T>(p, o, ou_sum(ss), t, h, lane, 32);
}

// One CTA per row. Gated values in shared memory by their place among the H * vdim values; a part's sum by the
// whole CTA where there are few parts, else by one warp.
template <typename T>
__global__ void __launch_bounds__(256) outer_part_norm_kernel(B200Outer p) {
  extern __shared__ float part_smem[];           // [H * vdim], [parts][8], [parts]
  pdl_wait();
  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, inner = p.H * p.V, n = p.H * p.vdim, ps = n / p.parts;
  const size_t t = blockIdx.x;
  float* sums = part_smem + ((n + 3) & ~3);
  float* inv = sums + p.parts * 8;
  const T* v = reinterpret_cast<const T*>(p.v) + t * p.ld;
  const T* z = reinterpret_cast<const T*>(p.gate) + t * p.ldg;
  const float* o = p.o + t * inner;
  const bool dense = p.V == p.vdim;
  for (int i = tid * 4; i < inner; i += 256 * 4) {
    const int h = (unsigned)i / (unsigned)p.V, c = i - h * p.V;
    const float d = p.skip[h];
    const float4 a = *reinterpret_cast<const float4*>(o + i), x = Ou4<T>::get(v + i), g = ou_silu(Ou4<T>::get(z + i));
    const float4 y = make_float4(fmaf(d, x.x, a.x) * g.x, fmaf(d, x.y, a.y) * g.y, fmaf(d, x.z, a.z) * g.z, fmaf(d, x.w, a.w) * g.w);
    if (dense) {
      *reinterpret_cast<float4*>(part_smem + i) = y;
    } else {
      const float e[4] = {y.x, y.y, y.z, y.w};
      for (int j = 0; j < 4; ++j)
        if (c + j < p.vdim) part_smem[h * p.vdim + c + j] = e[j];
    }
  }
  __syncthreads();
  if (p.parts < 8) {
    for (int g = 0; g < p.parts; ++g) {
      float ss = 0.f;
      for (int i = tid; i < ps; i += 256) ss = fmaf(part_smem[g * ps + i], part_smem[g * ps + i], ss);
      ss = ou_sum(ss);
      if (lane == 0) sums[g * 8 + warp] = ss;
    }
    __syncthreads();
    if (tid < p.parts) {
      float ss = 0.f;
      for (int w = 0; w < 8; ++w) ss += sums[tid * 8 + w];
      inv[tid] = p.out_scale / sqrtf(ss / (float)ps + p.eps);
    }
  } else {
    for (int g = warp; g < p.parts; g += 8) {
      float ss = 0.f;
      for (int i = lane; i < ps; i += 32) ss = fmaf(part_smem[g * ps + i], part_smem[g * ps + i], ss);
      ss = ou_sum(ss);
      if (lane == 0) inv[g] = p.out_scale / sqrtf(ss / (float)ps + p.eps);
    }
  }
  __syncthreads();
  T* out = reinterpret_cast<T*>(p.out) + t * p.ldo;
  if (dense && !(ps & 3)) {
    for (int i = tid * 4; i < inner; i += 256 * 4) {
      const float f = inv[(unsigned)i / (unsigned)ps];
      const float4 y = *reinterpret_cast<const float4*>(part_smem + i), w = *reinterpret_cast<const float4*>(p.norm_w + i);
      Ou4<T>::put(out + i, make_float4(y.x * f * w.x, y.y * f * w.y, y.z * f * w.z, y.w * f * w.w));
    }
  } else {
    for (int i = tid; i < inner; i += 256) {
      const int h = i / p.V, c = i - h * p.V, x = h * p.vdim + c;
      out[i] = T(c < p.vdim ? part_smem[x] * inv[x / ps] * p.norm_w[i] : 0.f);
    }
  }
}

static constexpr int kMaxSize = 1024;

bool outer_ok(const B200Outer* a) {
  return (a->kind == 0 || a->kind == 1) && a->H > 0 && a->G > 0 && a->H % a->G == 0 && a->D > 0 && a->V > 0 && !(a->D & 15) &&
         !(a->V & 15) && a->D <= kMaxSize && a->V <= kMaxSize && a->dim > 0 && a->vdim > 0 && a->dim <= a->D && a->vdim <= a->V &&
         !(a->ld & 3) && !(a->ldg & 3) && !(a->ldo & 3) && a->q && a->k && a->v && a->state && a->o && a->gate && a->norm_w && a->out &&
         (a->kind ? a->dt && a->dt_bias && a->A && a->skip && a->parts > 0 && a->H * a->vdim % a->parts == 0
                  : a->a1 && a->a2 && a->a2b && a->rank > 0 && !(a->rank & 15) && !(a->lda1 & 3) && a->H == a->G);
}

template <typename T, int KIND>
static cudaError_t launch_step(const B200Outer& a, int reqs, cudaStream_t stream) {
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
  const size_t smem = (size_t)(4 * a.D + a.V + slices * a.V) * 4;
  const dim3 grid(reqs, a.H);
  if (threads == 512)
    return rps <= 32 ? launch_pdl(outer_step_kernel<T, KIND, 32, 512>, grid, dim3(512), smem, stream, a, slices, rps)
                     : launch_pdl(outer_step_kernel<T, KIND, 0, 512>, grid, dim3(512), smem, stream, a, slices, rps);
  if (rps <= 8) return launch_pdl(outer_step_kernel<T, KIND, 8, 256>, grid, dim3(256), smem, stream, a, slices, rps);
  if (rps <= 16) return launch_pdl(outer_step_kernel<T, KIND, 16, 256>, grid, dim3(256), smem, stream, a, slices, rps);
  return launch_pdl(outer_step_kernel<T, KIND, 32, 256>, grid, dim3(256), smem, stream, a, slices, rps);
}

template <typename T>
static cudaError_t launch_parts(const B200Outer& a, size_t smem, cudaStream_t stream) {
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(outer_part_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  return launch_pdl(outer_part_norm_kernel<T>, dim3(a.rows.T), dim3(256), smem, stream, a);
}

}  // namespace b200

using namespace b200;

extern "C" {

// reqs: the first of them that are run here (the decode rows, or those and the portions).
int b200_outer_step(const B200Outer* a, int reqs, cudaStream_t stream) {
  if (reqs <= 0) return 0;
  if (!outer_ok(a)) return -1;
  if (a->H > 65535) return -4;
  cudaError_t e;
  if (a->kind == 0) e = a->f32 ? launch_step<float, 0>(*a, reqs, stream) : launch_step<bf16, 0>(*a, reqs, stream);
  else e = a->f32 ? launch_step<float, 1>(*a, reqs, stream) : launch_step<bf16, 1>(*a, reqs, stream);
  return e == cudaSuccess ? 0 : -2;
}

// What is left of norm and gate once b200_outer_step has run ``reqs`` requests and (chunks) b200_outer_chunk the portions.
int b200_outer_norm(const B200Outer* a, int reqs, int chunks, cudaStream_t stream) {
  if (a->rows.T <= 0) return 0;
  if (!outer_ok(a)) return -1;
  (void)reqs;
  if (a->kind == 1) {
    const size_t smem = ((size_t)a->H * a->vdim + 4 + (size_t)a->parts * 9) * 4;
    if (smem > 220 * 1024) return -4;
    return (a->f32 ? launch_parts<float>(*a, smem, stream) : launch_parts<bf16>(*a, smem, stream)) == cudaSuccess ? 0 : -2;
  }
  const int rows = chunks ? a->rows.T - a->rows.nd : 0;
  if (rows <= 0) return 0;
  if (a->V <= 128 && (long)rows * a->H < (1l << 31)) {
    const uint32_t items = (uint32_t)rows * a->H;
    const dim3 vgrid((items + 4 * kNormItems - 1) / (4 * kNormItems));
    return (a->f32 ? launch_pdl(outer_head_norm_vec_kernel<float>, vgrid, dim3(128), 0, stream, *a, a->rows.nd, items)
                   : launch_pdl(outer_head_norm_vec_kernel<bf16>, vgrid, dim3(128), 0, stream, *a, a->rows.nd, items)) == cudaSuccess ? 0 : -2;
  }
  const dim3 grid((unsigned)(((long)rows * a->H + 3) / 4));
  return (a->f32 ? launch_pdl(outer_head_norm_kernel<float>, grid, dim3(128), 0, stream, *a, a->rows.nd, rows)
                 : launch_pdl(outer_head_norm_kernel<bf16>, grid, dim3(128), 0, stream, *a, a->rows.nd, rows)) == cudaSuccess ? 0 : -2;
}

}  // extern "C"
