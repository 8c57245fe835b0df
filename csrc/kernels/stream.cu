// The fp32 residual stream of models that keep it in 32 bits, and true fp32 products (no reduced
// precision mode) for running such a model in 32 bits throughout.
//   stream_norm_kernel   embedding or residual update (+ expert outputs gathered per token, + norm of the
//                        update) + RMSNorm
//   gemm_f32_kernel      out = A W^T (+ bias), plain or per expert chunk
//   softcap_kernel      cap tanh(x / cap) of fp32 logits
//   clamped_gate_kernel, gated_act_kernel   activation of [gate | up] rows
#include "api.h"
#include "sm100.cuh"

namespace b200 {

template <typename T> struct Vec4;
template <> struct Vec4<float> {
  static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Vec4<__nv_bfloat16> {
  static __device__ __forceinline__ float4 load(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  }
};
__device__ __forceinline__ void add4(float4& x, float4 y) { x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w; }

static constexpr int kMaxPairs = 128;    // expert outputs per row

// One CTA per row; a thread keeps its four-value groups in registers between the two passes
// (kRegs groups), wider rows are read again from the stream.
template <typename T, int kRegs>
__global__ void __launch_bounds__(256) stream_norm_kernel(B200StreamNorm p, int* status) {
  __shared__ float red[8];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, nv = p.cols >> 2;
  float* s = p.stream + (size_t)t * p.lds;
  const T* src = nullptr;
  if (p.ids) {
    const int64_t id = reinterpret_cast<const int64_t*>(p.ids)[t];
    if (id >= 0 && id < p.vocab) src = reinterpret_cast<const T*>(p.table) + (size_t)id * p.cols;
    else if (threadIdx.x == 0 && status) atomicExch(status, (int)kErrBadArg);
  }
  // the row's pairs; ident rows (or nothing) stand for y where there is no expert output
  __shared__ const T* s_y[kMaxPairs];
  __shared__ float s_w[kMaxPairs];
  for (int x = threadIdx.x; x < p.k; x += blockDim.x) {
    const int32_t at = reinterpret_cast<const int32_t*>(p.pair_pos)[(size_t)t * p.k + x];
    s_y[x] = at >= 0 ? reinterpret_cast<const T*>(p.y) + (size_t)at * p.ldy
                               : p.ident ? reinterpret_cast<const T*>(p.ident) + (size_t)t * p.ldi : nullptr;
    s_w[x] = p.pair_w ? p.pair_w[(size_t)t * p.k + x] : 1.f;
  }
  if (p.k > 0) __syncthreads();
  float4 keep[kRegs], old[kRegs];        // update, then new stream; old stream (asked for ahead of the sums)
#pragma unroll
  for (int c = 0; c < kRegs; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i < nv && !p.ids) old[c] = Vec4<float>::load(s + i * 4);
  }
  auto row_sum = [&](float ss) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
    for (int w = 0; w < (int)(blockDim.x >> 5); ++w) ss += red[w];
    return ss;
  };
  auto sq = [](float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; };
  auto update = [&](int i) {             // what is added to the stream (or starts it)
    float4 v;
    if (p.ids) {
      v = src ? Vec4<T>::load(src + i * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
      v.x *= p.scale; v.y *= p.scale; v.z *= p.scale; v.w *= p.scale;
      return v;
    }
    v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.a) {
      if (p.a_f32) add4(v, Vec4<float>::load(reinterpret_cast<const float*>(p.a) + (size_t)t * p.lda + i * 4));
      else add4(v, Vec4<T>::load(reinterpret_cast<const T*>(p.a) + (size_t)t * p.lda + i * 4));
    }
    for (int j = 0; j < p.k; j += 4) {     // (four loads on the way at a time)
      float4 y[4];
#pragma unroll
      for (int x = 0; x < 4; ++x)
        y[x] = j + x < p.k && s_y[j + x] ? Vec4<T>::load(s_y[j + x] + i * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int x = 0; x < 4; ++x)
        if (j + x < p.k) {
          const float w = s_w[j + x];
          v.x = fmaf(w, y[x].x, v.x); v.y = fmaf(w, y[x].y, v.y); v.z = fmaf(w, y[x].z, v.z); v.w = fmaf(w, y[x].w, v.w);
        }
    }
    return v;
  };
  float post = 1.f;                      // 1 / rms of the update
  if (p.post_w) {
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < kRegs; ++c) {
      const int i = threadIdx.x + c * blockDim.x;
      if (i < nv) {
        keep[c] = update(i);
        ss += sq(keep[c]);
      }
    }
    for (int i = threadIdx.x + kRegs * blockDim.x; i < nv; i += blockDim.x) ss += sq(update(i));
    post = 1.f / sqrtf(row_sum(ss) / (float)p.width + p.eps);
    __syncthreads();                     // (red is used again)
  }
  auto value = [&](int i, float4 v, float4 before) {
    if (p.post_w) {
      const float4 w = Vec4<float>::load(p.post_w + i * 4);
      v.x *= post * (w.x + p.norm_offset); v.y *= post * (w.y + p.norm_offset);
      v.z *= post * (w.z + p.norm_offset); v.w *= post * (w.w + p.norm_offset);
    }
    if (!p.ids) {
      v.x *= p.mult; v.y *= p.mult; v.z *= p.mult; v.w *= p.mult;
      add4(v, before);
    }
    return v;
  };
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < kRegs; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i < nv) {
      keep[c] = value(i, p.post_w ? keep[c] : update(i), old[c]);
      Vec4<float>::store(s + i * 4, keep[c]);
      ss += sq(keep[c]);
    }
  }
  for (int i = threadIdx.x + kRegs * blockDim.x; i < nv; i += blockDim.x) {
    const float4 v = value(i, update(i), Vec4<float>::load(s + i * 4));
    Vec4<float>::store(s + i * 4, v);
    ss += sq(v);
  }
  const float inv = 1.f / sqrtf(row_sum(ss) / (float)p.width + p.eps);
  T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo;
  auto finish = [&](int i, float4 v) {
    const float4 w = Vec4<float>::load(p.norm_w + i * 4);
    Vec4<T>::store(out + i * 4, make_float4(v.x * inv * (w.x + p.norm_offset), v.y * inv * (w.y + p.norm_offset),
                                            v.z * inv * (w.z + p.norm_offset), v.w * inv * (w.w + p.norm_offset)));
  };
#pragma unroll
  for (int c = 0; c < kRegs; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i < nv) finish(i, keep[c]);
  }
  for (int i = threadIdx.x + kRegs * blockDim.x; i < nv; i += blockDim.x) finish(i, Vec4<float>::load(s + i * 4));
}

template <typename T>
static cudaError_t launch_stream_norm(const B200StreamNorm& a, int threads, cudaStream_t stream) {
  const int groups = (a.cols / 4 + threads - 1) / threads;
  const dim3 grid(a.T), block(threads);
  int* st = device_status_word();
  if (groups <= 1) return launch_pdl(stream_norm_kernel<T, 1>, grid, block, 0, stream, a, st);
  if (groups <= 2) return launch_pdl(stream_norm_kernel<T, 2>, grid, block, 0, stream, a, st);
  return launch_pdl(stream_norm_kernel<T, 4>, grid, block, 0, stream, a, st);
}

// ------------------------------------------------------------------------------------ fp32 products
struct F32Gemm {
  const float* A;
  const float* W;
  const float* bias;
  float* out;
  int lda, ldw, ldo, M, N, K;
  // batched (blockIdx.z): columns of A, rows of W, columns of out
  long long a_batch, w_batch, out_batch;
  // grouped: chunk c covers rows [row0[c], row0[c] + n[c]) of A / out with the matrix of expert[c]
  const int32_t* chunk_expert;
  const int32_t* chunk_row0;
  const int32_t* chunk_n;
  const int32_t* num_chunks;
  int act;
};

static constexpr int kFT = 64, kFK = 16;

// 64 x 64 tile, 256 threads of 4 x 4 outputs. Grouped: blockIdx.z = chunk, blockIdx.y = row tile in it.
__global__ void __launch_bounds__(256) gemm_f32_kernel(F32Gemm p) {
  __shared__ float sa[kFK][kFT + 4], sw[kFK][kFT + 4];
  pdl_wait();
  pdl_launch_dependents();
  const float* W = p.W;
  const float* A = p.A;
  float* out = p.out;
  int row_base = 0, rows = p.M;
  if (p.chunk_expert) {
    if ((int)blockIdx.z >= *p.num_chunks) return;
    W += (size_t)p.chunk_expert[blockIdx.z] * p.N * p.ldw;
    row_base = p.chunk_row0[blockIdx.z];
    rows = p.chunk_n[blockIdx.z];
  } else {
    A += blockIdx.z * p.a_batch;
    W += blockIdx.z * p.w_batch;
    out += blockIdx.z * p.out_batch;
  }
  const int m0 = blockIdx.y * kFT, n0 = blockIdx.x * kFT;
  if (m0 >= rows) return;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < p.K; k0 += kFK) {
    for (int x = threadIdx.x; x < kFT * kFK; x += 256) {
      const int r = x >> 4, k = x & 15;
      const bool kin = k0 + k < p.K;
      sa[k][r] = (kin && m0 + r < rows) ? A[(size_t)(row_base + m0 + r) * p.lda + k0 + k] : 0.f;
      sw[k][r] = (kin && n0 + r < p.N) ? W[(size_t)(n0 + r) * p.ldw + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kFK; ++k) {
      float a[4], w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sa[k][ty * 4 + i]; w[i] = sw[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= rows) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < p.N) out[(size_t)(row_base + m) * p.ldo + n] = act_epilogue<false>(acc[i][j] + (p.bias ? p.bias[n] : 0.f), p.act);
    }
  }
}

__global__ void __launch_bounds__(128)
    clamped_gate_kernel(const float* __restrict__ gu, float* out, const int32_t* total, int I, B200ClampedGate act) {
  pdl_wait();
  pdl_launch_dependents();
  const int row = blockIdx.x;
  if (row >= *total) return;
  const float w = act.row_w ? act.row_w[row] : 1.f;
  for (int i = threadIdx.x; i < I; i += blockDim.x) {
    const float g = fminf(gu[(size_t)row * 2 * I + i] * w, act.limit);
    const float u = fminf(fmaxf(gu[(size_t)row * 2 * I + I + i] * w, -act.limit), act.limit);
    out[(size_t)row * I + i] = g / (1.f + expf(-act.alpha * g)) * (u + act.up_offset);
  }
}

// out = act(gate) * up of fp32 rows [gate (I) | up (I)]. kind: 0 SiLU, 1 GELU-tanh, 2 GELU-erf.
__global__ void __launch_bounds__(128) gated_act_kernel(const float* gu, int ldg, float* out, int ldo, int I, int kind) {
  pdl_wait();
  pdl_launch_dependents();
  const float* g = gu + (size_t)blockIdx.x * ldg;
  for (int i = threadIdx.x; i < I; i += blockDim.x) {
    const float x = g[i];
    float a;
    if (kind == 0) a = x / (1.f + expf(-x));
    else if (kind == 1) a = 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
    else a = 0.5f * x * (1.f + erff(x * 0.7071067811865476f));
    out[(size_t)blockIdx.x * ldo + i] = a * g[I + i];
  }
}

// x = cap tanh(x / cap), as cap (1 - 2 / (1 + exp(2 x / cap))); near 0, where that cancels, by tanhf.
__global__ void __launch_bounds__(256) softcap_kernel(float* x, long long n4, long long n, float cap) {
  pdl_wait();
  pdl_launch_dependents();
  const float inv = 1.f / cap;
  auto f = [&](float v) {
    const float z = v * inv;
    return cap * (fabsf(z) < 0.5f ? tanhf(z) : 1.f - 2.f / (1.f + expf(2.f * z)));
  };
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i < n4) {
    float4 v = reinterpret_cast<float4*>(x)[i];
    v = make_float4(f(v.x), f(v.y), f(v.z), f(v.w));
    reinterpret_cast<float4*>(x)[i] = v;
  } else if (n4 * 4 + (i - n4) < n) {
    x[n4 * 4 + (i - n4)] = f(x[n4 * 4 + (i - n4)]);
  }
}

}  // namespace b200

using namespace b200;

extern "C" {

int b200_stream_norm(const B200StreamNorm* a, cudaStream_t stream) {
  if (a->T <= 0) return 0;
  if (!a->stream || !a->out || !a->norm_w || a->width <= 0 || a->cols < a->width || (a->cols & 7) || a->k < 0) return -1;
  if ((a->lds & 3) || (a->lda & 3) || (a->ldy & 3) || (a->ldi & 3) || (a->ldo & 3) || (a->ids && !a->table)) return -1;
  if (a->k > 0 && (!a->pair_pos || !a->y)) return -1;
  if (a->k > kMaxPairs) return -4;
  int threads = ((a->cols / 4 + 31) / 32) * 32;
  if (threads > 256) threads = 256;
  return (a->f32 ? launch_stream_norm<float>(*a, threads, stream) : launch_stream_norm<__nv_bfloat16>(*a, threads, stream)) ==
                 cudaSuccess ? 0 : -2;
}

int b200_gemm_f32(const void* A, int lda, const void* W, int ldw, void* out, int ldo, const void* bias, int M, int N,
                  int K, int act, cudaStream_t stream) {
  if (M <= 0 || N <= 0 || K <= 0) return 0;
  F32Gemm p{(const float*)A, (const float*)W, (const float*)bias, (float*)out, lda, ldw, ldo, M, N, K,
            0, 0, 0, nullptr, nullptr, nullptr, nullptr, act};
  dim3 grid((N + kFT - 1) / kFT, (M + kFT - 1) / kFT);
  if (grid.y > 65535) return -4;
  return launch_pdl(gemm_f32_kernel, grid, dim3(256), 0, stream, p) == cudaSuccess ? 0 : -2;
}

// out[m, b * out_batch + n] = sum_k A[m, b * a_batch + k] W[b * N + n, k]
int b200_gemm_f32_batched(const void* A, int lda, int a_batch, const void* W, int ldw, void* out, int ldo,
                          long long out_batch, int M, int N, int K, int batch, cudaStream_t stream) {
  if (M <= 0 || N <= 0 || K <= 0 || batch <= 0) return 0;
  F32Gemm p{(const float*)A, (const float*)W, nullptr, (float*)out, lda, ldw, ldo, M, N, K,
            a_batch, (long long)N * ldw, out_batch, nullptr, nullptr, nullptr, nullptr, 0};
  dim3 grid((N + kFT - 1) / kFT, (M + kFT - 1) / kFT, batch);
  if (grid.y > 65535 || grid.z > 65535) return -4;
  return launch_pdl(gemm_f32_kernel, grid, dim3(256), 0, stream, p) == cudaSuccess ? 0 : -2;
}

int b200_softcap_f32(void* x, long long n, float cap, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (!(cap > 0.f)) return -1;
  const long long n4 = ((uintptr_t)x & 15) ? 0 : n / 4, items = n4 + (n - n4 * 4);
  return launch_pdl(softcap_kernel, dim3((unsigned)((items + 255) / 256)), dim3(256), 0, stream, (float*)x, n4, n, cap) ==
                 cudaSuccess ? 0 : -2;
}

int b200_moe_grouped_gemm_f32(const void* xs, int max_rows, const void* W, int E, int N, int K, void* out,
                              const void* chunk_expert, const void* chunk_row0, const void* chunk_n, const void* meta,
                              int max_chunks, cudaStream_t stream) {
  return b200_moe_grouped_gemm_f32_act(xs, max_rows, W, E, N, K, out, chunk_expert, chunk_row0, chunk_n, meta, max_chunks, 0,
                                       stream);
}

int b200_moe_grouped_gemm_f32_act(const void* xs, int max_rows, const void* W, int E, int N, int K, void* out,
                                  const void* chunk_expert, const void* chunk_row0, const void* chunk_n, const void* meta,
                                  int max_chunks, int act, cudaStream_t stream) {
  if (max_rows <= 0) return 0;
  if (max_chunks > 65535) return -4;
  F32Gemm p{(const float*)xs, (const float*)W, nullptr, (float*)out, K, K, N, max_rows, N, K,
            0, 0, 0, (const int32_t*)chunk_expert, (const int32_t*)chunk_row0, (const int32_t*)chunk_n,
            (const int32_t*)meta + 3 * E + 1, act};
  dim3 grid((N + kFT - 1) / kFT, 256 / kFT, max_chunks);     // a chunk has at most 256 rows
  return launch_pdl(gemm_f32_kernel, grid, dim3(256), 0, stream, p) == cudaSuccess ? 0 : -2;
}

int b200_gated_act_f32(const void* gate_up, int ldg, void* out, int ldo, int T, int I, int kind, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (I <= 0 || kind < 0 || kind > 2) return -1;
  return launch_pdl(gated_act_kernel, dim3(T), dim3(128), 0, stream, (const float*)gate_up, ldg, (float*)out, ldo, I,
                    kind) == cudaSuccess ? 0 : -2;
}

int b200_clamped_gate_f32(const void* gate_up, void* out, const void* meta, int E, int max_rows, int I,
                          const B200ClampedGate* act, cudaStream_t stream) {
  if (max_rows <= 0) return 0;
  if (!act || I <= 0) return -1;
  return launch_pdl(clamped_gate_kernel, dim3(max_rows), dim3(128), 0, stream, (const float*)gate_up, (float*)out,
                    (const int32_t*)meta + 2 * E, I, *act) == cudaSuccess ? 0 : -2;
}

}  // extern "C"
