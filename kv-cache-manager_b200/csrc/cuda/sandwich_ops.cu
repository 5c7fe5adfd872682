// Kernels of blocks whose sublayers are normalised on both sides (x <- x + post(sublayer(pre(x)))) and of
// the parts such designs bring along.  All arithmetic is float whatever the storage type T of the rows
// that go on to a matrix product; the residual stream x and every sublayer's output y are float.
//
//   embed_scaled    x[t] = table[id[t]] * scale (and a copy for parts that read the embedding later)
//   norm_post_pre   x += wb * y / rms(y)   (if y);   out = T(wn * x / rms(x))   (if out; optionally of gathered rows)
//                   -- the norm that closes one sublayer and the norm that opens the next in one pass; y is a float row, the
//                   sum of two normalised branches, or the weighted sum over a row's experts, formed in the same pass
//   poly_norm_act   out = T(a N(z) + b N(z^2) + c N(z^3) + e), N(v) = v / rms(v) over a row, powers element-wise
//   concat_cast     out[t] = [T(a[t]) | T(b[t])]
//   add_bias_rows   x[t] += bias
//   softcap_rows    x <- cap * tanh(x / cap)
//   rotate_heads    turns pairs of the first `n` dimensions of every head of a row by sign * position * freq
//   gla_prepare     q *= qscale;  z <- sigmoid(z + bias)^(1/tau)  evaluated as exp(logsigmoid(z + bias) / tau)
//
// rms(v) = sqrt(mean(v^2) + eps).  Weights are given as the multipliers themselves, in float.
#include "common.cuh"
#include "pdl.cuh"

namespace kvcm {

template <typename T>
__global__ void __launch_bounds__(256)
embed_scaled_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ x,
                    float* __restrict__ keep, int H, int vocab, float scale) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* src = table + size_t(id) * H;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float v = ldf(src + i) * scale;
    x[size_t(t) * H + i] = v;
    if (keep) keep[size_t(t) * H + i] = v;
  }
}

// Four values a thread and access (H % 4 == 0 and 16-byte aligned rows); as many threads as a row has float4s, at most 512.
__device__ __forceinline__ void st4(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void st4(bf16* p, float a, float b, float c, float d) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  uint2 u;
  u.x = *reinterpret_cast<const unsigned*>(&lo);
  u.y = *reinterpret_cast<const unsigned*>(&hi);
  *reinterpret_cast<uint2*>(p) = u;
}

// What a sublayer returned, y:
//   kYNone     nothing is pending
//   kYDense    one float row
//   kYJoined   the sum of two branches, each first divided by its own root mean square: w0 * y0 / rms(y0) + w1 * y1 / rms(y1)
//   kYExperts  the weighted sum over a row's experts, sum_k wt[row, k] y[place of (row, k)]
enum { kYNone = 0, kYDense = 1, kYJoined = 2, kYExperts = 3 };
struct NormPostPreParams {
  float* x;
  const float* y; const float* y1; const float* w0; const float* w1; float eps_join;
  const int* place; const float* wt; int top;
  const float* wb; const float* wn; void* out; const int* rows;
  int H; float eps;
};

__device__ __forceinline__ void load_cols(float (&v)[4], const float* p) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void load_cols(float (&v)[1], const float* p) { v[0] = *p; }
template <typename T> __device__ __forceinline__ void store_cols(T* p, const float (&v)[4]) { st4(p, v[0], v[1], v[2], v[3]); }
template <typename T> __device__ __forceinline__ void store_cols(T* p, const float (&v)[1]) { stf(p, v[0]); }

// Two block-wide sums at once, with one barrier (`scratch`, 32 pairs, is not used again by the launch).
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  if (lane == 0) scratch[warp] = make_float2(a, b);
  __syncthreads();
  float2 t = lane < nwarps ? scratch[lane] : make_float2(0.f, 0.f);
  t.x = warp_sum(t.x);
  t.y = warp_sum(t.y);
  return t;
}

// One block a row, V neighbouring values a thread and access (V = 4: H % 4 == 0 and 16-byte aligned rows); every global
// load of the row is asked for before the first sum, and the values wait in shared memory ([y | x], joined: [y0 | x | y1]).
template <typename T, int V, int MODE>
__global__ void __launch_bounds__(512)
norm_post_pre_kernel(NormPostPreParams p) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[33];
  __shared__ float2 scratch2[32];
  pdl_launch_dependents();
  const int H = p.H, tid = V * threadIdx.x, step = V * blockDim.x;
  const int r = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  float* xs = row + H;
  float* ys = row + 2 * H;
  float* xr = p.x + size_t(r) * H;
  pdl_wait();
  float sa = 0.f, sb = 0.f;
  for (int i = tid; i < H; i += step) {
    float x[V], y[V];
    load_cols(x, xr + i);
    if constexpr (MODE == kYNone) {
#pragma unroll
      for (int e = 0; e < V; ++e) sb = fmaf(x[e], x[e], sb);
    } else if constexpr (MODE == kYExperts) {
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = 0.f;
      for (int k = 0; k < p.top; ++k) {
        float a[V];
        load_cols(a, p.y + size_t(p.place[size_t(r) * p.top + k]) * H + i);
        const float w = p.wt[size_t(r) * p.top + k];
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = fmaf(w, a[e], y[e]);
      }
    } else {
      load_cols(y, p.y + size_t(r) * H + i);
    }
    if constexpr (MODE == kYJoined) {
      float z[V];
      load_cols(z, p.y1 + size_t(r) * H + i);
#pragma unroll
      for (int e = 0; e < V; ++e) sb = fmaf(z[e], z[e], sb);
      store_cols(ys + i, z);
    }
    if constexpr (MODE != kYNone) {
#pragma unroll
      for (int e = 0; e < V; ++e) sa = fmaf(y[e], y[e], sa);
      store_cols(row + i, y);
    }
    store_cols(xs + i, x);
  }
  float s2 = sb;
  if constexpr (MODE != kYNone) {
    if constexpr (MODE == kYJoined) {
      const float2 t = block_sum2(sa, sb, scratch2);
      const float i0 = 1.f / sqrtf(t.x / float(H) + p.eps_join), i1 = 1.f / sqrtf(t.y / float(H) + p.eps_join);
      sa = 0.f;
      for (int i = tid; i < H; i += step) {
        float y[V], z[V], w0[V], w1[V];
        load_cols(w0, p.w0 + i);
        load_cols(w1, p.w1 + i);
        load_cols(y, row + i);
        load_cols(z, ys + i);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          y[e] = w0[e] * (y[e] * i0) + w1[e] * (z[e] * i1);
          sa = fmaf(y[e], y[e], sa);
        }
        store_cols(row + i, y);
      }
    }
    const float inv = 1.f / sqrtf(block_sum(sa, scratch) / float(H) + p.eps);
    s2 = 0.f;
    for (int i = tid; i < H; i += step) {
      float x[V], y[V], w[V];
      load_cols(w, p.wb + i);
      load_cols(x, xs + i);
      load_cols(y, row + i);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        x[e] = x[e] + w[e] * (y[e] * inv);
        s2 = fmaf(x[e], x[e], s2);
      }
      store_cols(xs + i, x);
      if (!p.rows) store_cols(xr + i, x);
    }
    if (!p.out) return;
  }
  const float inv2 = 1.f / sqrtf(block_sum(s2, scratch) / float(H) + p.eps);
  T* o = reinterpret_cast<T*>(p.out) + size_t(blockIdx.x) * H;
  for (int i = tid; i < H; i += step) {
    float x[V], w[V];
    load_cols(w, p.wn + i);
    load_cols(x, xs + i);
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = w[e] * (x[e] * inv2);
    store_cols(o + i, x);
  }
}

// The same for rows whose float4s fit NQ a thread: the row stays in registers, the weights (which no launch of the step
// writes) are asked for before the wait, and every sum costs one barrier.
template <typename T, int NQ, int MODE>
__global__ void __launch_bounds__(512)
norm_post_pre_regs_kernel(NormPostPreParams p) {
  __shared__ float2 scratch[3][32];
  pdl_launch_dependents();
  const int H = p.H;
  const int r = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  float* xr = p.x + size_t(r) * H;
  float x[NQ][4], y[NQ][4], wb[NQ][4], wn[NQ][4];
  float z[MODE == kYJoined ? NQ : 1][4], w0[MODE == kYJoined ? NQ : 1][4], w1[MODE == kYJoined ? NQ : 1][4];
  auto at = [&](int q) { return 4 * int(threadIdx.x + q * blockDim.x); };
#pragma unroll
  for (int q = 0; q < NQ; ++q) {
    if (at(q) >= H) continue;
    if constexpr (MODE != kYNone) load_cols(wb[q], p.wb + at(q));
    if (p.out) load_cols(wn[q], p.wn + at(q));
    if constexpr (MODE == kYJoined) {
      load_cols(w0[q], p.w0 + at(q));
      load_cols(w1[q], p.w1 + at(q));
    }
  }
  pdl_wait();
#pragma unroll
  for (int q = 0; q < NQ; ++q) {
#pragma unroll
    for (int e = 0; e < 4; ++e) x[q][e] = y[q][e] = 0.f;
    if constexpr (MODE == kYJoined) z[q][0] = z[q][1] = z[q][2] = z[q][3] = 0.f;
    if (at(q) >= H) continue;
    load_cols(x[q], xr + at(q));
    if constexpr (MODE == kYDense || MODE == kYJoined) load_cols(y[q], p.y + size_t(r) * H + at(q));
    if constexpr (MODE == kYJoined) load_cols(z[q], p.y1 + size_t(r) * H + at(q));
  }
  if constexpr (MODE == kYExperts) {
#pragma unroll 4
    for (int k = 0; k < p.top; ++k) {
      const float* src = p.y + size_t(p.place[size_t(r) * p.top + k]) * H;
      const float w = p.wt[size_t(r) * p.top + k];
#pragma unroll
      for (int q = 0; q < NQ; ++q) {
        if (at(q) >= H) continue;
        float a[4];
        load_cols(a, src + at(q));
#pragma unroll
        for (int e = 0; e < 4; ++e) y[q][e] = fmaf(w, a[e], y[q][e]);
      }
    }
  }
  float s2 = 0.f;
  if constexpr (MODE != kYNone) {
    float sa = 0.f, sb = 0.f;
    if constexpr (MODE == kYJoined) {
#pragma unroll
      for (int q = 0; q < NQ; ++q)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          sa = fmaf(y[q][e], y[q][e], sa);
          sb = fmaf(z[q][e], z[q][e], sb);
        }
      const float2 t = block_sum2(sa, sb, scratch[0]);
      const float i0 = 1.f / sqrtf(t.x / float(H) + p.eps_join), i1 = 1.f / sqrtf(t.y / float(H) + p.eps_join);
#pragma unroll
      for (int q = 0; q < NQ; ++q)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (at(q) < H) y[q][e] = w0[q][e] * (y[q][e] * i0) + w1[q][e] * (z[q][e] * i1);
      sa = 0.f;
    }
#pragma unroll
    for (int q = 0; q < NQ; ++q)
#pragma unroll
      for (int e = 0; e < 4; ++e) sa = fmaf(y[q][e], y[q][e], sa);
    const float inv = 1.f / sqrtf(block_sum2(sa, 0.f, scratch[1]).x / float(H) + p.eps);
#pragma unroll
    for (int q = 0; q < NQ; ++q) {
      if (at(q) >= H) continue;
#pragma unroll
      for (int e = 0; e < 4; ++e) x[q][e] = x[q][e] + wb[q][e] * (y[q][e] * inv);
      if (!p.rows) store_cols(xr + at(q), x[q]);
    }
    if (!p.out) return;
  }
#pragma unroll
  for (int q = 0; q < NQ; ++q)
#pragma unroll
    for (int e = 0; e < 4; ++e) s2 = fmaf(x[q][e], x[q][e], s2);
  const float inv2 = 1.f / sqrtf(block_sum2(s2, 0.f, scratch[2]).x / float(H) + p.eps);
  T* o = reinterpret_cast<T*>(p.out) + size_t(blockIdx.x) * H;
#pragma unroll
  for (int q = 0; q < NQ; ++q) {
    if (at(q) >= H) continue;
#pragma unroll
    for (int e = 0; e < 4; ++e) x[q][e] = wn[q][e] * (x[q][e] * inv2);
    store_cols(o + at(q), x[q]);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
poly_norm_act_kernel(const float* __restrict__ z, int ldz, const float* __restrict__ coef, T* __restrict__ out, int F,
                     float eps) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[33];
  pdl_launch_dependents();
  pdl_wait();
  const float* zr = z + size_t(blockIdx.x) * ldz;
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  for (int i = threadIdx.x; i < F; i += blockDim.x) {
    const float v = zr[i];
    row[i] = v;
    const float v2 = v * v, v3 = v2 * v;
    s2 += v2;
    s4 = fmaf(v2, v2, s4);
    s6 = fmaf(v3, v3, s6);
  }
  s2 = block_sum(s2, scratch);
  s4 = block_sum(s4, scratch);
  s6 = block_sum(s6, scratch);
  const float n = float(F);
  const float a = coef[0] / sqrtf(s2 / n + eps), b = coef[1] / sqrtf(s4 / n + eps), c = coef[2] / sqrtf(s6 / n + eps);
  const float e = coef[3];
  T* o = out + size_t(blockIdx.x) * F;
  for (int i = threadIdx.x; i < F; i += blockDim.x) {
    const float v = row[i], v2 = v * v;
    stf(o + i, a * v + b * v2 + c * (v2 * v) + e);
  }
}

template <typename T>
__global__ void __launch_bounds__(512)
poly_norm_act_vec_kernel(const float* __restrict__ z, int ldz, const float* __restrict__ coef, T* __restrict__ out, int F,
                         float eps) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[33];
  pdl_launch_dependents();
  pdl_wait();
  const float* zr = z + size_t(blockIdx.x) * ldz;
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  for (int i = 4 * threadIdx.x; i < F; i += 4 * blockDim.x) {
    const float4 q = *reinterpret_cast<const float4*>(zr + i);
    *reinterpret_cast<float4*>(row + i) = q;
    const float e[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float v2 = e[k] * e[k], v3 = v2 * e[k];
      s2 += v2;
      s4 = fmaf(v2, v2, s4);
      s6 = fmaf(v3, v3, s6);
    }
  }
  s2 = block_sum(s2, scratch);
  s4 = block_sum(s4, scratch);
  s6 = block_sum(s6, scratch);
  const float n = float(F);
  const float a = coef[0] / sqrtf(s2 / n + eps), b = coef[1] / sqrtf(s4 / n + eps), c = coef[2] / sqrtf(s6 / n + eps);
  const float e0 = coef[3];
  T* o = out + size_t(blockIdx.x) * F;
  for (int i = 4 * threadIdx.x; i < F; i += 4 * blockDim.x) {
    const float4 q = *reinterpret_cast<const float4*>(row + i);
    const float x2 = q.x * q.x, y2 = q.y * q.y, z2 = q.z * q.z, w2 = q.w * q.w;
    st4(o + i, a * q.x + b * x2 + c * (x2 * q.x) + e0, a * q.y + b * y2 + c * (y2 * q.y) + e0,
        a * q.z + b * z2 + c * (z2 * q.z) + e0, a * q.w + b * w2 + c * (w2 * q.w) + e0);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
concat_cast_kernel(const float* __restrict__ a, const float* __restrict__ b, T* __restrict__ out, int H) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    stf(out + t * 2 * H + i, a[t * H + i]);
    stf(out + t * 2 * H + H + i, b[t * H + i]);
  }
}

__global__ void __launch_bounds__(256)
add_bias_rows_kernel(float* __restrict__ x, const float* __restrict__ bias, int H) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  for (int i = threadIdx.x; i < H; i += blockDim.x) x[t * H + i] += bias[i];
}

__global__ void __launch_bounds__(256)
softcap_rows_kernel(float* __restrict__ x, long long n, float cap) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) x[i] = cap * tanhf(x[i] / cap);
}

// One block a row, a warp a head at a time.
template <typename T>
__global__ void __launch_bounds__(128)
rotate_heads_kernel(T* __restrict__ x, int ldx, const int* __restrict__ positions, const float* __restrict__ inv_freq,
                    int n, int interleaved, float sign, int nh, int HD) {
  extern __shared__ __align__(16) float cs[];        // n/2 cosines, n/2 sines
  pdl_launch_dependents();
  const int half = n / 2;
  const float pos = float(positions[blockIdx.x]);
  for (int j = threadIdx.x; j < half; j += blockDim.x) {
    float sn, c;
    sincosf(pos * inv_freq[j], &sn, &c);
    cs[j] = c;
    cs[half + j] = sign * sn;
  }
  pdl_wait();
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  for (int h = warp; h < nh; h += nwarps) {
    T* v = x + size_t(blockIdx.x) * ldx + size_t(h) * HD;
    for (int j = lane; j < half; j += 32) {
      const int ia = interleaved ? 2 * j : j, ib = interleaved ? 2 * j + 1 : j + half;
      float a, b;
      rotate_pair(ldf(v + ia), ldf(v + ib), cs[j], cs[half + j], a, b);
      stf(v + ia, a);
      stf(v + ib, b);
    }
  }
}

// qkv rows [.. q: n_q floats at q_base ..]; z rows [heads*dk] become the decays.
__global__ void __launch_bounds__(256)
gla_prepare_kernel(float* __restrict__ qkv, int channels, int q_base, int n_q, float qscale, float* __restrict__ z,
                   const float* __restrict__ bias, int n_z, float inv_tau) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  for (int i = threadIdx.x; i < n_q; i += blockDim.x) qkv[t * channels + q_base + i] *= qscale;
  for (int i = threadIdx.x; i < n_z; i += blockDim.x) {
    const float v = z[t * n_z + i] + (bias ? bias[i] : 0.f);
    const float ls = fminf(v, 0.f) - log1pf(expf(-fabsf(v)));      // log sigmoid(v)
    z[t * n_z + i] = expf(ls * inv_tau);
  }
}

}  // namespace kvcm

using namespace kvcm;

// Threads of a four-values-a-thread kernel over rows of n values: one float4 each, between 64 and 512.
static int vec_threads(int n) {
  const int t = ((n / 4) + 31) / 32 * 32;
  return t < 64 ? 64 : (t > 512 ? 512 : t);
}
template <typename... P>
static bool aligned16(const P*... p) {
  return (((reinterpret_cast<uintptr_t>(p)) | ...) & 15) == 0;
}

#define KVCM_EMBED_SCALED_ARGS const int *ids, const void *table, float *x, float *keep, int rows, int H, int vocab, float scale, void *stream
KVCM_API int kvcm_embed_scaled_f32(KVCM_EMBED_SCALED_ARGS) {
  if (rows == 0) return 0;
  return pdl_launch(embed_scaled_kernel<float>, dim3(rows), dim3(256), 0, (cudaStream_t)stream, ids, (const float*)table, x,
                    keep, H, vocab, scale);
}
KVCM_API int kvcm_embed_scaled_bf16(KVCM_EMBED_SCALED_ARGS) {
  if (rows == 0) return 0;
  return pdl_launch(embed_scaled_kernel<bf16>, dim3(rows), dim3(256), 0, (cudaStream_t)stream, ids, (const bf16*)table, x,
                    keep, H, vocab, scale);
}

template <typename T, int V, int MODE>
static int launch_norm_post_pre_as(const NormPostPreParams& p, int rows, cudaStream_t s) {
  if constexpr (V == 4) {
    const int quads = p.H / 4;
    if (quads <= 512 && (rows < 256 || quads < 128))     // (many rows: fewer, longer threads and more rows at a time)
      return pdl_launch(norm_post_pre_regs_kernel<T, 1, MODE>, dim3(rows), dim3((quads + 31) / 32 * 32), 0, s, p);
    if (quads <= 1024)
      return pdl_launch(norm_post_pre_regs_kernel<T, 2, MODE>, dim3(rows), dim3((quads + 63) / 64 * 32), 0, s, p);
  }
  const size_t smem = size_t(p.H) * (MODE == kYJoined ? 3 : 2) * sizeof(float);
  if (smem > 200 * 1024) return KVCM_ERR_UNSUPPORTED;
  static size_t configured = 0;
  if (smem > 40 * 1024 && smem > configured) {          // (the kernel's static shared memory counts against the 48 KB too)
    const cudaError_t e = cudaFuncSetAttribute(norm_post_pre_kernel<T, V, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    if (e != cudaSuccess) return int(e);
    configured = smem;
  }
  return pdl_launch(norm_post_pre_kernel<T, V, MODE>, dim3(rows), dim3(V == 4 ? vec_threads(p.H) : 256), smem, s, p);
}
template <typename T>
static int launch_norm_post_pre(const NormPostPreParams& p, int rows, cudaStream_t s) {
  if (rows == 0) return 0;
  const bool joined = p.y1 != nullptr, experts = p.place != nullptr;
  if ((p.y && !p.wb) || (p.out && !p.wn) || (!p.y && (!p.out || joined || experts)) || (p.rows && !p.out) || (joined && (experts || !p.w0 || !p.w1)) ||
      (experts && (!p.wt || p.top < 1)))
    return KVCM_ERR_UNSUPPORTED;
  const bool vec = p.H % 4 == 0 && aligned16(p.x, p.y, p.y1, p.w0, p.w1, p.wb, p.wn) && aligned16(static_cast<const char*>(p.out));
#define KVCM_NORM_MODE(MODE) return vec ? launch_norm_post_pre_as<T, 4, MODE>(p, rows, s) : launch_norm_post_pre_as<T, 1, MODE>(p, rows, s)
  if (!p.y) KVCM_NORM_MODE(kYNone);
  if (joined) KVCM_NORM_MODE(kYJoined);
  if (experts) KVCM_NORM_MODE(kYExperts);
  KVCM_NORM_MODE(kYDense);
#undef KVCM_NORM_MODE
}
// y1 (with w0, w1, eps_join): y is the first of two branches that are normalised and summed; place, wt, top: y holds the
// experts' outputs in the order of the sorted pairs.
#define KVCM_NORM_POST_PRE_ARGS                                                                                           \
  float *x, const float *y, const float *y1, const float *w0, const float *w1, float eps_join, const int *place,          \
      const float *wt, int top, const float *wb, const float *wn, void *out, const int *rows_idx, int rows, int H, float eps, void *stream
static NormPostPreParams norm_post_pre_params(KVCM_NORM_POST_PRE_ARGS) {
  (void)rows; (void)stream;
  return NormPostPreParams{x, y, y1, w0, w1, eps_join, place, wt, top, wb, wn, out, rows_idx, H, eps};
}
KVCM_API int kvcm_norm_post_pre_f32(KVCM_NORM_POST_PRE_ARGS) {
  return launch_norm_post_pre<float>(norm_post_pre_params(x, y, y1, w0, w1, eps_join, place, wt, top, wb, wn, out, rows_idx, rows, H, eps, stream), rows, (cudaStream_t)stream);
}
KVCM_API int kvcm_norm_post_pre_bf16(KVCM_NORM_POST_PRE_ARGS) {
  return launch_norm_post_pre<bf16>(norm_post_pre_params(x, y, y1, w0, w1, eps_join, place, wt, top, wb, wn, out, rows_idx, rows, H, eps, stream), rows, (cudaStream_t)stream);
}

template <typename T>
static int launch_poly_norm(const float* z, int ldz, const float* coef, void* out, int rows, int F, float eps, cudaStream_t s) {
  if (rows == 0) return 0;
  const size_t smem = size_t(F) * sizeof(float);
  if (smem > 200 * 1024) return KVCM_ERR_UNSUPPORTED;
  if (F % 4 == 0 && ldz % 4 == 0 && aligned16(z, out)) {
    if (smem > 40 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(poly_norm_act_vec_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
      if (e != cudaSuccess) return int(e);
    }
    return pdl_launch(poly_norm_act_vec_kernel<T>, dim3(rows), dim3(vec_threads(F)), smem, s, z, ldz, coef, (T*)out, F, eps);
  }
  if (smem > 40 * 1024) {                               // (the kernel's static shared memory counts against the 48 KB too)
    const cudaError_t e = cudaFuncSetAttribute(poly_norm_act_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    if (e != cudaSuccess) return int(e);
  }
  return pdl_launch(poly_norm_act_kernel<T>, dim3(rows), dim3(256), smem, s, z, ldz, coef, (T*)out, F, eps);
}
KVCM_API int kvcm_poly_norm_act_f32(const float* z, int ldz, const float* coef, void* out, int rows, int F, float eps, void* stream) {
  return launch_poly_norm<float>(z, ldz, coef, out, rows, F, eps, (cudaStream_t)stream);
}
KVCM_API int kvcm_poly_norm_act_bf16(const float* z, int ldz, const float* coef, void* out, int rows, int F, float eps, void* stream) {
  return launch_poly_norm<bf16>(z, ldz, coef, out, rows, F, eps, (cudaStream_t)stream);
}

KVCM_API int kvcm_concat_cast_f32(const float* a, const float* b, void* out, int rows, int H, void* stream) {
  if (rows == 0) return 0;
  return pdl_launch(concat_cast_kernel<float>, dim3(rows), dim3(256), 0, (cudaStream_t)stream, a, b, (float*)out, H);
}
KVCM_API int kvcm_concat_cast_bf16(const float* a, const float* b, void* out, int rows, int H, void* stream) {
  if (rows == 0) return 0;
  return pdl_launch(concat_cast_kernel<bf16>, dim3(rows), dim3(256), 0, (cudaStream_t)stream, a, b, (bf16*)out, H);
}

KVCM_API int kvcm_add_bias_rows(float* x, const float* bias, int rows, int H, void* stream) {
  if (rows == 0) return 0;
  return pdl_launch(add_bias_rows_kernel, dim3(rows), dim3(256), 0, (cudaStream_t)stream, x, bias, H);
}

KVCM_API int kvcm_softcap_rows(float* x, long long n, float cap, void* stream) {
  if (n == 0) return 0;
  if (!(cap > 0.f)) return KVCM_ERR_UNSUPPORTED;
  softcap_rows_kernel<<<unsigned((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(x, n, cap);
  return KVCM_LAUNCH_RESULT();
}

#define KVCM_ROTATE_HEADS_ARGS void *x, int ldx, const int *positions, const float *inv_freq, int n, int interleaved, float sign, int rows, int nh, int HD, void *stream
template <typename T>
static int launch_rotate_heads(KVCM_ROTATE_HEADS_ARGS) {
  if (rows == 0 || n == 0) return 0;
  if (n % 2 || n > HD) return KVCM_ERR_UNSUPPORTED;
  return pdl_launch(rotate_heads_kernel<T>, dim3(rows), dim3(128), size_t(n) * sizeof(float), (cudaStream_t)stream, (T*)x, ldx,
                    positions, inv_freq, n, interleaved, sign, nh, HD);
}
KVCM_API int kvcm_rotate_heads_f32(KVCM_ROTATE_HEADS_ARGS) {
  return launch_rotate_heads<float>(x, ldx, positions, inv_freq, n, interleaved, sign, rows, nh, HD, stream);
}
KVCM_API int kvcm_rotate_heads_bf16(KVCM_ROTATE_HEADS_ARGS) {
  return launch_rotate_heads<bf16>(x, ldx, positions, inv_freq, n, interleaved, sign, rows, nh, HD, stream);
}

KVCM_API int kvcm_gla_prepare(float* qkv, int channels, int q_base, int n_q, float qscale, float* z, const float* bias, int n_z,
                              float tau, int rows, void* stream) {
  if (rows == 0) return 0;
  if (!(tau > 0.f)) return KVCM_ERR_UNSUPPORTED;
  return pdl_launch(gla_prepare_kernel, dim3(rows), dim3(256), 0, (cudaStream_t)stream, qkv, channels, q_base, n_q, qscale, z,
                    bias, n_z, 1.f / tau);
}
