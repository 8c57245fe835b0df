// The fp32 stream of models whose sublayers read short convolutions of a normed stream.
//
//   embed_pairs_kernel   token and token-pair embeddings, norm in equal parts, each request's last token
//   norm_conv_kernel     stream update (+ expert outputs gathered per token), norm in equal parts, and up to two causal
//                        convolutions over the normed rows with carried rows: one CTA per part of the width and run of
//                        kRun rows, which norms the taps - 1 rows ahead of its run once more
//
// The stream is read from one buffer and written to another, so that a run may look at its neighbours' rows.
#include "api.h"
#include "sm100.cuh"

namespace b200 {

typedef __nv_bfloat16 bf16;

static constexpr int kRun = 16;          // rows of a portion that one CTA walks
static constexpr int kBatch = 4;         // rows on the way at a time
static constexpr int kPairs = 64;        // expert outputs per row
static constexpr int kAhead = 4;         // of a row on the way at a time

// VEC values in memory (Raw) and as floats
template <typename T, int VEC> struct Vals;
template <> struct Vals<float, 4> {
  typedef float4 Raw;
  static __device__ __forceinline__ void open(Raw r, float* v) { *reinterpret_cast<float4*>(v) = r; }
  static __device__ __forceinline__ void get(const float* p, float* v) { *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void put(float* p, const float* v) { *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(v); }
};
template <> struct Vals<bf16, 4> {
  typedef uint2 Raw;
  static __device__ __forceinline__ void open(Raw u, float* v) {
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
  static __device__ __forceinline__ void get(const bf16* p, float* v) { open(*reinterpret_cast<const uint2*>(p), v); }
  static __device__ __forceinline__ void put(bf16* p, const float* v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  }
};
template <> struct Vals<float, 1> {
  typedef float Raw;
  static __device__ __forceinline__ void open(Raw r, float* v) { *v = r; }
  static __device__ __forceinline__ void get(const float* p, float* v) { *v = *p; }
  static __device__ __forceinline__ void put(float* p, const float* v) { *p = *v; }
};
template <> struct Vals<bf16, 1> {
  typedef bf16 Raw;
  static __device__ __forceinline__ void open(Raw r, float* v) { *v = __bfloat162float(r); }
  static __device__ __forceinline__ void get(const bf16* p, float* v) { *v = __bfloat162float(*p); }
  static __device__ __forceinline__ void put(bf16* p, const float* v) { *p = __float2bfloat16(*v); }
};

// ------------------------------------------------------------------------------------ embeddings
// One CTA per row. The CTA of a portion's first row reads the request's last token and replaces it.
template <typename T>
__global__ void __launch_bounds__(256) embed_pairs_kernel(B200EmbedPairs p, int* status) {
  extern __shared__ float row_smem[];            // [cols] values, [groups] 1 / rms
  __shared__ long long s_pair;
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const B200Rows& R = p.rows;
  const int64_t* ids = reinterpret_cast<const int64_t*>(p.ids);
  const int64_t id = ids[t];
  if (tid == 0 && p.bigram) {
    int req = t, at = 0, len = 1;
    if (t >= R.nd) {
      int lo = 0, hi = R.num_prefills - 1;
      while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (R.q_start[mid] <= t - R.nd) lo = mid; else hi = mid - 1;
      }
      req = R.nd + lo;
      at = t - R.nd - R.q_start[lo];
      len = R.q_start[lo + 1] - R.q_start[lo];
    }
    const int slot = R.slots[req];
    long long before = -1;
    if (at > 0) before = ids[t - 1];
    else if (slot >= 0 && R.seq_lens[req] > len) before = p.prev[slot];
    if (at == 0 && slot >= 0) p.prev[slot] = ids[t + len - 1];
    s_pair = before < 0 ? p.buckets : (long long)(((unsigned long long)before * p.mul_prev + (unsigned long long)id * p.mul_cur) %
                                                  (unsigned long long)p.buckets);
  }
  __syncthreads();
  const bool known = id >= 0 && id < p.vocab;
  if (!known && tid == 0 && status) atomicExch(status, (int)kErrBadArg);
  const T* e = reinterpret_cast<const T*>(p.table) + (size_t)(known ? id : 0) * p.cols;
  const T* b = p.bigram ? reinterpret_cast<const T*>(p.bigram) + (size_t)s_pair * p.cols : nullptr;
  for (int i = tid * 4; i < p.cols; i += blockDim.x * 4) {
    float v[4], w[4] = {0.f, 0.f, 0.f, 0.f};
    Vals<T, 4>::get(e + i, v);
    if (b) Vals<T, 4>::get(b + i, w);
#pragma unroll
    for (int x = 0; x < 4; ++x) v[x] = fmaf(known ? v[x] : 0.f, p.scale, w[x]);
    Vals<float, 4>::put(row_smem + i, v);
  }
  __syncthreads();
  // every warp sums a slice of every part
  const int gs = p.width / p.groups, nw = blockDim.x >> 5;
  float* part = row_smem + p.cols;               // [groups][warps], then [groups]
  for (int g = 0; g < p.groups; ++g) {
    float ss = 0.f;
    if (!(gs & 3))
      for (int i = tid * 4; i < gs; i += blockDim.x * 4) {
        float v[4];
        Vals<float, 4>::get(row_smem + g * gs + i, v);
#pragma unroll
        for (int x = 0; x < 4; ++x) ss = fmaf(v[x], v[x], ss);
      }
    else
      for (int i = tid; i < gs; i += blockDim.x) ss = fmaf(row_smem[g * gs + i], row_smem[g * gs + i], ss);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (lane == 0) part[g * nw + warp] = ss;
  }
  __syncthreads();
  float* inv = part + p.groups * nw;
  for (int g = tid; g < p.groups; g += blockDim.x) {
    float ss = 0.f;
    for (int w = 0; w < nw; ++w) ss += part[g * nw + w];
    inv[g] = 1.f / sqrtf(ss / (float)gs + p.eps);
  }
  __syncthreads();
  float* out = p.stream + (size_t)t * p.lds;
  if (!(gs & 3)) {
    for (int i = tid * 4; i < p.cols; i += blockDim.x * 4) {
      float v[4] = {0.f, 0.f, 0.f, 0.f}, w[4];
      if (i < p.width) {
        const float f = inv[i / gs];
        Vals<float, 4>::get(row_smem + i, v);
        Vals<float, 4>::get(p.norm_w + i, w);
#pragma unroll
        for (int x = 0; x < 4; ++x) v[x] *= f * w[x];
      }
      Vals<float, 4>::put(out + i, v);
    }
    return;
  }
  for (int i = tid; i < p.cols; i += blockDim.x) out[i] = i < p.width ? row_smem[i] * inv[i / gs] * p.norm_w[i] : 0.f;
}

// ------------------------------------------------------------------- update, norm, convolutions
// grid (runs, parts). VEC consecutive values a thread at a time, NV of those; TAPS 0: any number, carried rows of the run in
// shared memory and taps read from memory. PAIRS: with expert outputs. MT: most threads.
template <typename T, int VEC, int NV, int TAPS, bool PAIRS, int MT>
__global__ void __launch_bounds__(MT, MT > 128 ? 1 : PAIRS ? 4 : 5) norm_conv_kernel(B200NormConv p) {
  extern __shared__ float4 nc_smem[];            // PAIRS: [rows][pairs] rows of y, weights; TAPS 0: [taps - 1][NV][threads][VEC]
  __shared__ float red[kBatch][16];
  pdl_wait();
  pdl_launch_dependents();
  const int tid = threadIdx.x, nt = blockDim.x, warp = tid >> 5, lane = tid & 31, taps = TAPS ? TAPS : p.taps;
  const B200Rows& R = p.rows;
  int req, row0, n, at, len;             // first row, rows, their offset in the portion, the portion's length
  if ((int)blockIdx.x < R.nd) {
    req = row0 = blockIdx.x;
    n = len = 1;
    at = 0;
  } else {
    const int u = blockIdx.x - R.nd, tile = u / (128 / kRun);
    const int r = R.tile_req[tile], b = R.q_start[r];
    at = R.tile_q0[tile] + (u % (128 / kRun)) * kRun;
    len = R.q_start[r + 1] - b;
    if (at >= len) return;
    req = R.nd + r;
    row0 = R.nd + b + at;
    n = min(kRun, len - at);
  }
  const int gs = p.width / p.groups, base = blockIdx.y * gs, first = row0 - at;      // the portion's first row
  const int slot = R.slots[req];
  const bool init = slot >= 0 && R.seq_lens[req] > len;
  bool on[NV];
  int col[NV];
#pragma unroll
  for (int c = 0; c < NV; ++c) {
    const int i = (c * nt + tid) * VEC;
    on[c] = i < gs;
    col[c] = base + (on[c] ? i : 0);
  }
  // the expert outputs of every row that this CTA looks at: its run with the taps - 1 rows ahead, and the portion's last taps - 1
  // (no output: weight 0, and some row that is there)
  const int k4 = PAIRS ? (p.k + kAhead - 1) / kAhead * kAhead : 0, ahead = at == 0 ? 0 : taps - 1;
  const int run = ahead + n, tail = at == 0 && len > n ? taps - 1 : 0;
  int32_t* s_y = reinterpret_cast<int32_t*>(nc_smem);                  // [kRun + 2 (taps - 1)][k4]
  float* s_w = reinterpret_cast<float*>(s_y + (kRun + 2 * (taps - 1)) * k4);
  if (PAIRS) {
    for (int i = tid; i < (run + tail) * k4; i += nt) {
      const int r = i / k4, j = i - r * k4, pos = r < run ? at - ahead + r : len - tail + (r - run);
      const size_t pair = (size_t)(first + pos) * p.k + min(j, p.k - 1);
      const int32_t y = reinterpret_cast<const int32_t*>(p.pair_pos)[pair];
      s_y[i] = max(y, 0);
      s_w[i] = y >= 0 && j < p.k ? p.pair_w[pair] : 0.f;
    }
    __syncthreads();
  }
  // Rows pos .. pos + count - 1 of the portion over their rms; those of this run (keep) also go to dst.
  auto normed = [&](int pos, int count, bool keep, float (&x)[kBatch][NV][VEC]) {
#pragma unroll
    for (int r = 0; r < kBatch; ++r)
#pragma unroll
      for (int c = 0; c < NV; ++c) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[r][c][e] = 0.f;
        if (r < count && on[c]) Vals<float, VEC>::get(p.src + (size_t)(first + pos + r) * p.lds + col[c], x[r][c]);
      }
    if (p.a) {
#pragma unroll
      for (int r = 0; r < kBatch; ++r)
#pragma unroll
        for (int c = 0; c < NV; ++c)
          if (r < count && on[c]) {
            float a[VEC];
            Vals<float, VEC>::get(p.a + (size_t)(first + pos + r) * p.lda + col[c], a);
#pragma unroll
            for (int e = 0; e < VEC; ++e) x[r][c][e] += a[e];
          }
    }
    if (PAIRS) {
      const int e0 = (keep ? pos - (at - ahead) : run + pos - (len - tail)) * k4;
      const T* y0 = reinterpret_cast<const T*>(p.y);
      constexpr int AH = NV * VEC <= 4 ? kAhead : 1;
      for (int j0 = 0; j0 < k4; j0 += AH) {      // (the loads of AH outputs of every row are on the way at a time)
        typename Vals<T, VEC>::Raw y[AH][kBatch][NV];
#pragma unroll
        for (int r = 0; r < kBatch; ++r)
          if (r < count) {
#pragma unroll
            for (int j = 0; j < AH; ++j) {
              const T* from = y0 + (size_t)s_y[e0 + r * k4 + j0 + j] * p.ldy;
#pragma unroll
              for (int c = 0; c < NV; ++c) y[j][r][c] = *reinterpret_cast<const typename Vals<T, VEC>::Raw*>(from + col[c]);
            }
          }
#pragma unroll
        for (int r = 0; r < kBatch; ++r)
          if (r < count) {
#pragma unroll
            for (int j = 0; j < AH; ++j) {
              const float w = s_w[e0 + r * k4 + j0 + j];
#pragma unroll
              for (int c = 0; c < NV; ++c) {
                float v[VEC];
                Vals<T, VEC>::open(y[j][r][c], v);
#pragma unroll
                for (int e = 0; e < VEC; ++e) x[r][c][e] = on[c] ? fmaf(w, v[e], x[r][c][e]) : 0.f;
              }
            }
          }
      }
    }
#pragma unroll
    for (int r = 0; r < kBatch; ++r) {
      float ss = 0.f;
#pragma unroll
      for (int c = 0; c < NV; ++c) {
        if (keep && p.dst && r < count && pos + r >= at && on[c])
          Vals<float, VEC>::put(p.dst + (size_t)(first + pos + r) * p.lds + col[c], x[r][c]);
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss = fmaf(x[r][c][e], x[r][c][e], ss);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (lane == 0) red[r][warp] = ss;
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < kBatch; ++r) {
      float ss = 0.f;
      for (int w = 0; w < (nt >> 5); ++w) ss += red[r][w];
      const float inv = 1.f / sqrtf(ss / (float)gs + p.eps);
#pragma unroll
      for (int c = 0; c < NV; ++c)
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[r][c][e] *= inv;
    }
    __syncthreads();                             // (red is used again)
  };

  float wt[TAPS ? 2 * TAPS : 1][NV][VEC], hist[TAPS > 1 ? TAPS - 1 : 1][NV][VEC];
  if (TAPS) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int c = 0; c < NV; ++c) {
        Vals<float, VEC>::get(p.w1 + (size_t)j * p.cols + col[c], wt[j][c]);
        if (p.out2) Vals<float, VEC>::get(p.w2 + (size_t)j * p.cols + col[c], wt[TAPS + j][c]);
      }
  }
  float* mine = s_w + (kRun + 2 * (taps - 1)) * k4 + tid * VEC;   // entry j, piece c: mine + (j * NV + c) * nt * VEC
  const int step = nt * VEC;
  auto carried = [&](int i, int c, float* v) {   // entry i of the state
    if (init && on[c]) {
      Vals<float, VEC>::get(p.state + ((size_t)slot * (taps - 1) + i) * p.cols + col[c], v);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = 0.f;
    }
  };
  auto push = [&](int c, const float* v) {       // the newest row of the history
    if (TAPS) {
#pragma unroll
      for (int j = 0; j + 2 < TAPS; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) hist[j][c][e] = hist[j + 1][c][e];
      if (TAPS > 1)
#pragma unroll
        for (int e = 0; e < VEC; ++e) hist[TAPS > 1 ? TAPS - 2 : 0][c][e] = v[e];
    } else {
      for (int j = 0; j + 2 < taps; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) mine[(j * NV + c) * step + e] = mine[((j + 1) * NV + c) * step + e];
      if (taps > 1)
#pragma unroll
        for (int e = 0; e < VEC; ++e) mine[((taps - 2) * NV + c) * step + e] = v[e];
    }
  };
  // rows ahead of the run: of the portion itself (a run starts at a multiple of kRun >= taps - 1), else carried ones
  if (at == 0) {
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      if (TAPS) {
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) carried(j, c, hist[j][c]);
      } else {
        for (int j = 0; j + 1 < taps; ++j) carried(j, c, mine + (j * NV + c) * step);
      }
    }
  }
  T* out1 = reinterpret_cast<T*>(p.out1);
  T* out2 = reinterpret_cast<T*>(p.out2);
  for (int pos = at == 0 ? 0 : at - (taps - 1); pos < at + n; pos += kBatch) {
    const int count = min(kBatch, at + n - pos);
    float x[kBatch][NV][VEC];
    normed(pos, count, true, x);
#pragma unroll
    for (int r = 0; r < kBatch; ++r) {
      if (r >= count) break;
      const size_t to = (size_t)(first + pos + r) * p.ldo;
#pragma unroll
      for (int c = 0; c < NV; ++c) {
        if (pos + r >= at && on[c]) {
          float y1[VEC], y2[VEC];
#pragma unroll
          for (int e = 0; e < VEC; ++e) y1[e] = y2[e] = 0.f;
          if (TAPS) {
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
              const float* v = j + 1 < TAPS ? hist[j + 1 < TAPS ? j : 0][c] : x[r][c];
#pragma unroll
              for (int e = 0; e < VEC; ++e) {
                y1[e] = fmaf(wt[j][c][e], v[e], y1[e]);
                if (p.out2) y2[e] = fmaf(wt[TAPS ? TAPS + j : 0][c][e], v[e], y2[e]);
              }
            }
          } else {
            for (int j = 0; j < taps; ++j)
#pragma unroll
              for (int e = 0; e < VEC; ++e) {
                const float v = j + 1 < taps ? mine[(j * NV + c) * step + e] : x[r][c][e];
                y1[e] = fmaf(p.w1[(size_t)j * p.cols + col[c] + e], v, y1[e]);
                if (p.out2) y2[e] = fmaf(p.w2[(size_t)j * p.cols + col[c] + e], v, y2[e]);
              }
          }
          Vals<T, VEC>::put(out1 + to + col[c], y1);
          if (p.out2) Vals<T, VEC>::put(out2 + to + col[c], y2);
        }
        push(c, x[r][c]);
      }
      if (blockIdx.y == gridDim.y - 1 && pos + r >= at)        // (padding meets zero weights and has to be finite)
        for (int i = p.width + tid; i < p.cols; i += nt) {
          const float zero = 0.f;
          Vals<T, 1>::put(out1 + to + i, &zero);
          if (p.out2) Vals<T, 1>::put(out2 + to + i, &zero);
        }
    }
  }
  // The first run hands on the portion's last rows, after its own look at the carried ones.
  if (taps <= 1 || at > 0 || slot < 0) return;
  float* st = p.state + (size_t)slot * (taps - 1) * p.cols;
  if (len <= n) {
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      if (!on[c]) continue;
      if (TAPS) {
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) Vals<float, VEC>::put(st + (size_t)j * p.cols + col[c], hist[j][c]);
      } else {
        for (int j = 0; j + 1 < taps; ++j) Vals<float, VEC>::put(st + (size_t)j * p.cols + col[c], mine + (j * NV + c) * step);
      }
    }
    return;
  }
  for (int j = 0; j + 1 < taps; j += kBatch) {
    const int count = min(kBatch, taps - 1 - j);
    float x[kBatch][NV][VEC];
    normed(len - (taps - 1) + j, count, false, x);
#pragma unroll
    for (int r = 0; r < kBatch; ++r)
#pragma unroll
      for (int c = 0; c < NV; ++c)
        if (r < count && on[c]) Vals<float, VEC>::put(st + (size_t)(j + r) * p.cols + col[c], x[r][c]);
  }
}

template <typename T, int VEC, int NV, int TAPS, bool PAIRS, int MT>
static int run_norm_conv(const B200NormConv& a, int threads, cudaStream_t stream) {
  const dim3 grid(a.rows.nd + a.rows.num_tiles * (128 / kRun), a.groups);
  const size_t k4 = PAIRS ? (a.k + kAhead - 1) / kAhead * kAhead : 0;
  const size_t smem = (kRun + 2 * (a.taps - 1)) * k4 * 8 + (TAPS ? 0 : (size_t)(a.taps - 1) * NV * VEC * threads * 4);
  if (smem > 160 * 1024) return -4;
  if (!TAPS) {
    static PerDeviceOnce once;
    if (once.first())
      cudaFuncSetAttribute(norm_conv_kernel<T, VEC, NV, TAPS, PAIRS, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
  }
  return launch_pdl(norm_conv_kernel<T, VEC, NV, TAPS, PAIRS, MT>, grid, dim3(threads), smem, stream, a) == cudaSuccess ? 0 : -2;
}
template <typename T, int VEC, int NV, int TAPS>
static int pick_pairs(const B200NormConv& a, int threads, cudaStream_t stream) {
  if constexpr (TAPS > 0 && NV == 1)
    if (threads <= 128)
      return a.k ? run_norm_conv<T, VEC, NV, TAPS, true, 128>(a, threads, stream) : run_norm_conv<T, VEC, NV, TAPS, false, 128>(a, threads, stream);
  return a.k ? run_norm_conv<T, VEC, NV, TAPS, true, 512>(a, threads, stream) : run_norm_conv<T, VEC, NV, TAPS, false, 512>(a, threads, stream);
}
template <typename T, int VEC, int NV>
static int pick_taps(const B200NormConv& a, int threads, cudaStream_t stream) {
  if constexpr (NV <= 2 && VEC == 4) {
    if (a.taps == 1) return pick_pairs<T, VEC, NV, 1>(a, threads, stream);
    if (a.taps == 2) return pick_pairs<T, VEC, NV, 2>(a, threads, stream);
    if (a.taps == 3) return pick_pairs<T, VEC, NV, 3>(a, threads, stream);
    if (a.taps == 4) return pick_pairs<T, VEC, NV, 4>(a, threads, stream);
  }
  return pick_pairs<T, VEC, NV, 0>(a, threads, stream);
}
template <typename T>
static int pick_width(const B200NormConv& a, cudaStream_t stream) {
  const int gs = a.width / a.groups;
  auto threads = [](int n) { return n >= 512 ? 512 : (n + 31) / 32 * 32; };
  if (gs % 4 == 0) {
    const int n = gs / 4;
    if (n <= 512) return pick_taps<T, 4, 1>(a, threads(n), stream);
    if (n <= 1024) return pick_taps<T, 4, 2>(a, threads((n + 1) / 2), stream);
    if (n <= 2048) return pick_taps<T, 4, 4>(a, threads((n + 3) / 4), stream);
    return -4;
  }
  if (gs <= 512) return pick_taps<T, 1, 1>(a, threads(gs), stream);
  if (gs <= 4096) return pick_taps<T, 1, 8>(a, threads((gs + 7) / 8), stream);
  return -4;
}

}  // namespace b200

using namespace b200;

extern "C" {

int b200_embed_pairs(const B200EmbedPairs* a, cudaStream_t stream) {
  if (a->rows.T <= 0) return 0;
  if (!a->stream || !a->ids || !a->table || !a->norm_w || a->width <= 0 || a->cols < a->width || (a->cols & 7) || a->groups <= 0 ||
      a->width % a->groups || (a->lds & 3) || (a->bigram && (!a->prev || a->buckets <= 0 || a->mul_prev < 0 || a->mul_cur < 0)))
    return -1;
  const size_t smem = ((size_t)a->cols + (size_t)a->groups * 9) * 4;
  if (smem > 200 * 1024) return -4;
  int* st = device_status_word();
  static PerDeviceOnce once;
  if (once.first()) {
    cudaFuncSetAttribute(embed_pairs_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    cudaFuncSetAttribute(embed_pairs_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  }
  return (a->f32 ? launch_pdl(embed_pairs_kernel<float>, dim3(a->rows.T), dim3(256), smem, stream, *a, st)
                 : launch_pdl(embed_pairs_kernel<bf16>, dim3(a->rows.T), dim3(256), smem, stream, *a, st)) == cudaSuccess ? 0 : -2;
}

int b200_norm_conv(const B200NormConv* a, cudaStream_t stream) {
  if (a->rows.nd + a->rows.num_tiles <= 0) return 0;
  if (!a->src || !a->w1 || !a->out1 || (a->out2 && !a->w2) || a->width <= 0 || a->cols < a->width || (a->cols & 7) || a->groups <= 0 ||
      a->width % a->groups || (a->lds & 3) || (a->lda & 3) || (a->ldy & 3) || (a->ldo & 3) || a->dst == a->src || a->taps < 1 ||
      a->taps > kRun + 1 || (a->taps > 1 && !a->state) || a->k < 0 || (a->k > 0 && (!a->y || !a->pair_pos || !a->pair_w)))
    return -1;
  if (a->k > kPairs || a->groups > 65535) return -4;
  return a->f32 ? pick_width<float>(*a, stream) : pick_width<bf16>(*a, stream);
}

}  // extern "C"
