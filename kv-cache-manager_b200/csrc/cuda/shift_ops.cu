// The row-wise kernel in front of a layer whose mixer and feed-forward read the same residual stream through
// norms of their own, and whose mixer mixes every row with the row before it (token shift):
//
//   x'  = x + s0 p0 + s1 p1 + s2 p2 + sum_k wt[row, k] y[place of (row, k)]        what the layer before left pending:
//                                  up to three float tensors, and the weighted sum over a row's experts
//   h   = w1 * x' / sqrt(mean(x'^2) + eps1)
//   out1 = h + (h_before - h) * shift        h_before: the h of the same request's row before this one, zeros at its
//                                            first token; without `shift`, out1 = h
//   out2 = w2 * x' / sqrt(mean(x'^2) + eps2)                                        (optional)
//
// h_before of a portion's first row is what the request's state row kept ([slots, D] float: the h of the last token
// computed so far, zeros at the start); of every other row it is formed again from the row before.  x' goes to a
// tensor of its own, so a block may read any row of x.  A block takes R rows, and with them the row before its first:
// all of them are loaded at once and share one reduction.  The state of a request is read and written by ONE block,
// the one that holds the request's first row of the step (it forms the h of the request's last row too, wherever
// that lies): no other block can overtake its read.
//
// With `rows` the outputs are formed for the listed rows only and x' is not stored (final norm).
// Everything is float; a row's result does not depend on its place in the batch.
#include "common.cuh"
#include "pdl.cuh"

namespace kvcm {

struct NormPairParams {
  const float* x; float* x_out;                      // x_out null: x' is not stored
  const float* p0; const float* p1; const float* p2;
  float s0, s1, s2;
  const float* ey; const int* place; const float* wt; int top;      // experts' outputs [rows * top, D] (ey null: none)
  const float* w1; float eps1; void* out1;
  const float* w2; float eps2; void* out2;           // out2 null: none
  const float* shift;                                // null: no shift
  float* state; long long state_stride;
  const int* row_seq; const int* seq_q_start; const int* seq_q_len; const int* seq_state_slot;
  const int* rows;                                   // null, or the rows to form
  int n, D;
};

template <int V> struct Cols;                        // V neighbouring columns
template <> struct Cols<4> {
  float v[4];
  static __device__ __forceinline__ Cols load(const float* p) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    return {{a.x, a.y, a.z, a.w}};
  }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
  __device__ __forceinline__ void store(bf16* p) const {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<const uint32_t*>(&a);
    raw.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
  }
};
template <> struct Cols<1> {
  float v[1];
  static __device__ __forceinline__ Cols load(const float* p) { return {{*p}}; }
  template <typename T> __device__ __forceinline__ void store(T* p) const { stf(p, v[0]); }
};

constexpr int kNormPairThreads = 512;
constexpr int kNormPairMaxRows = 4;

// Slots of a block: 0 = the row before its first (when a shift needs it), 1..R = its rows, R + 1 = the last row of a
// request that starts in this block and ends in a later one (its h becomes the request's state).
template <typename T, int V, int R>
__global__ void __launch_bounds__(kNormPairThreads, 2)
norm_pair_kernel(NormPairParams p) {
  constexpr int S = R + 2;
  extern __shared__ __align__(16) float vals[];      // [S][D], then (with experts) S * top weights and S * top places
  __shared__ float part[kNormPairThreads / 32][S];
  __shared__ float inv1[S], inv2[S];
  __shared__ int src[S], slot_of[S], first_of[S], last_of[S];
  pdl_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarps = blockDim.x >> 5;
  const int D = p.D, row0 = blockIdx.x * R;
  if (tid < S) {                                     // (the batch's integers: no kernel of the step writes them)
    int s = -1, slot = -1, first = 0, last = 0;
    const int row = row0 + tid - 1;
    if (tid >= 1 && tid <= R && row < p.n) s = p.rows ? p.rows[row] : row;
    if (p.shift) {
      if (s >= 0) {
        const int q = p.row_seq[s], q0 = p.seq_q_start[q];
        slot = p.seq_state_slot[q];
        first = s == q0;
        last = s == q0 + p.seq_q_len[q] - 1 && q0 >= row0;          // the state is this block's to write
      } else if (tid == 0 && row0 > 0 && p.seq_q_start[p.row_seq[row0]] != row0) {
        s = row0 - 1;
      } else if (tid == R + 1) {
        const int end = min(row0 + R, p.n);                          // the request of the block's last row
        const int q = p.row_seq[end - 1], q0 = p.seq_q_start[q], tail = q0 + p.seq_q_len[q] - 1;
        if (q0 >= row0 && tail >= end) { s = tail; slot = p.seq_state_slot[q]; }
      }
    }
    src[tid] = s; slot_of[tid] = slot; first_of[tid] = first; last_of[tid] = last;
  }
  float* ewt = vals + size_t(S) * D;
  int* eplace = reinterpret_cast<int*>(ewt + S * p.top);
  __syncthreads();
  pdl_wait();
  if (p.ey) {
    for (int i = tid; i < S * p.top; i += blockDim.x) {
      const int s = src[i / p.top];
      const size_t at = size_t(max(s, 0)) * p.top + i % p.top;
      ewt[i] = s >= 0 ? p.wt[at] : 0.f;
      eplace[i] = s >= 0 ? p.place[at] : 0;
    }
    __syncthreads();
  }

  float ss[S];
#pragma unroll
  for (int j = 0; j < S; ++j) ss[j] = 0.f;
  for (int i = V * tid; i < D; i += V * blockDim.x) {
    Cols<V> c[S];
#pragma unroll
    for (int j = 0; j < S; ++j) {
      if (src[j] < 0) continue;
      c[j] = Cols<V>::load(p.x + size_t(src[j]) * D + i);
    }
    auto add = [&](const float* y, float scale) {
#pragma unroll
      for (int j = 0; j < S; ++j) {
        if (src[j] < 0) continue;
        const Cols<V> a = Cols<V>::load(y + size_t(src[j]) * D + i);
#pragma unroll
        for (int e = 0; e < V; ++e) c[j].v[e] = fmaf(scale, a.v[e], c[j].v[e]);
      }
    };
    if (p.p0) add(p.p0, p.s0);
    if (p.p1) add(p.p1, p.s1);
    if (p.p2) add(p.p2, p.s2);
    if (p.ey) {
      for (int k = 0; k < p.top; ++k)
#pragma unroll
        for (int j = 0; j < S; ++j) {
          if (src[j] < 0) continue;
          const Cols<V> a = Cols<V>::load(p.ey + size_t(eplace[j * p.top + k]) * D + i);
          const float w = ewt[j * p.top + k];
#pragma unroll
          for (int e = 0; e < V; ++e) c[j].v[e] = fmaf(w, a.v[e], c[j].v[e]);
        }
    }
#pragma unroll
    for (int j = 0; j < S; ++j) {
      if (src[j] < 0) continue;
      c[j].store(vals + size_t(j) * D + i);
      if (j >= 1 && j <= R && p.x_out) c[j].store(p.x_out + size_t(src[j]) * D + i);
#pragma unroll
      for (int e = 0; e < V; ++e) ss[j] = fmaf(c[j].v[e], c[j].v[e], ss[j]);
    }
  }
#pragma unroll
  for (int j = 0; j < S; ++j) {
    const float t = warp_sum(ss[j]);
    if (lane == 0) part[warp][j] = t;
  }
  __syncthreads();
  if (tid < S) {
    float t = 0.f;
    for (int w = 0; w < nwarps; ++w) t += part[w][tid];
    t /= float(D);
    inv1[tid] = 1.f / sqrtf(t + p.eps1);
    inv2[tid] = 1.f / sqrtf(t + p.eps2);
  }
  __syncthreads();

  T* out1 = reinterpret_cast<T*>(p.out1);
  T* out2 = reinterpret_cast<T*>(p.out2);
  for (int i = V * tid; i < D; i += V * blockDim.x) {
    const Cols<V> w1 = Cols<V>::load(p.w1 + i);
    Cols<V> w2 = {}, sh = {}, before = {};
    if (out2) w2 = Cols<V>::load(p.w2 + i);
    if (p.shift) {
      sh = Cols<V>::load(p.shift + i);
      if (src[0] >= 0) {
        const Cols<V> c = Cols<V>::load(vals + i);
#pragma unroll
        for (int e = 0; e < V; ++e) before.v[e] = c.v[e] * inv1[0] * w1.v[e];
      }
    }
#pragma unroll
    for (int j = 1; j <= R; ++j) {
      if (src[j] < 0) continue;
      const int row = row0 + j - 1;
      const Cols<V> c = Cols<V>::load(vals + size_t(j) * D + i);
      Cols<V> h, o;
#pragma unroll
      for (int e = 0; e < V; ++e) h.v[e] = c.v[e] * inv1[j] * w1.v[e];
      if (p.shift) {
        float* st = slot_of[j] >= 0 ? p.state + slot_of[j] * p.state_stride + i : nullptr;
        if (first_of[j]) {
          if (st) before = Cols<V>::load(st);
          else before = {};
        }
#pragma unroll
        for (int e = 0; e < V; ++e) o.v[e] = fmaf(before.v[e] - h.v[e], sh.v[e], h.v[e]);
        if (last_of[j] && st) h.store(st);           // (this thread has read the request's old state of these columns)
        before = h;
        o.store(out1 + size_t(row) * D + i);
      } else {
        h.store(out1 + size_t(row) * D + i);
      }
      if (out2) {
#pragma unroll
        for (int e = 0; e < V; ++e) o.v[e] = c.v[e] * inv2[j] * w2.v[e];
        o.store(out2 + size_t(row) * D + i);
      }
    }
    if (p.shift && src[R + 1] >= 0 && slot_of[R + 1] >= 0) {
      const Cols<V> c = Cols<V>::load(vals + size_t(R + 1) * D + i);
      Cols<V> h;
#pragma unroll
      for (int e = 0; e < V; ++e) h.v[e] = c.v[e] * inv1[R + 1] * w1.v[e];
      h.store(p.state + slot_of[R + 1] * p.state_stride + i);
    }
  }
}

static size_t norm_pair_smem(const NormPairParams& p, int R) {
  return size_t(R + 2) * (size_t(p.D) * sizeof(float) + (p.ey ? size_t(p.top) * 8 : 0));
}

template <typename T, int V, int R>
static int launch_norm_pair_as(const NormPairParams& p, cudaStream_t s) {
  const size_t smem = norm_pair_smem(p, R);
  static size_t configured = 0;
  if (smem > 40 * 1024 && smem > configured) {      // (the static arrays come on top)
    const cudaError_t e = cudaFuncSetAttribute(norm_pair_kernel<T, V, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    if (e != cudaSuccess) return int(e);
    configured = smem;
  }
  const int threads = min(kNormPairThreads, max(64, (p.D / V + 31) / 32 * 32));
  return pdl_launch(norm_pair_kernel<T, V, R>, dim3((p.n + R - 1) / R), dim3(threads), smem, s, p);
}

template <typename T>
static int launch_norm_pair(const NormPairParams& p, cudaStream_t s) {
  if (p.n == 0) return 0;
  if (p.D < 1 || norm_pair_smem(p, 1) > 200 * 1024) return KVCM_ERR_UNSUPPORTED;
  auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = (p.D % 4) == 0 && (p.state_stride % 4) == 0 && aligned(p.x) && aligned(p.x_out) && aligned(p.p0) && aligned(p.p1) &&
                   aligned(p.p2) && aligned(p.ey) && aligned(p.w1) && aligned(p.w2) && aligned(p.out1) && aligned(p.out2) &&
                   aligned(p.shift) && aligned(p.state);
  // Many rows: four a block (the row before the first is formed again: a quarter more reads, mostly from L2), else one.
  const bool four = p.shift && p.n >= 512 && norm_pair_smem(p, kNormPairMaxRows) <= 110 * 1024;
  if (vec) return four ? launch_norm_pair_as<T, 4, kNormPairMaxRows>(p, s) : launch_norm_pair_as<T, 4, 1>(p, s);
  return four ? launch_norm_pair_as<T, 1, kNormPairMaxRows>(p, s) : launch_norm_pair_as<T, 1, 1>(p, s);
}

}  // namespace kvcm

using namespace kvcm;

#define KVCM_NORM_PAIR_ARGS                                                                                              \
  const float *x, float *x_out, const float *p0, float s0, const float *p1, float s1, const float *p2, float s2,         \
      const float *ey, const int *place, const float *wt, int top, const float *w1, float eps1, void *out1,              \
      const float *w2, float eps2, void *out2, const float *shift, float *state, long long state_stride,                 \
      const int *row_seq, const int *seq_q_start, const int *seq_q_len, const int *seq_state_slot, const int *rows,      \
      int n, int D, void *stream
static NormPairParams norm_pair_params(KVCM_NORM_PAIR_ARGS) {
  (void)stream;
  NormPairParams p;
  p.x = x; p.x_out = x_out; p.p0 = p0; p.p1 = p1; p.p2 = p2; p.s0 = s0; p.s1 = s1; p.s2 = s2;
  p.ey = ey; p.place = place; p.wt = wt; p.top = ey ? top : 0;
  p.w1 = w1; p.eps1 = eps1; p.out1 = out1; p.w2 = w2; p.eps2 = eps2; p.out2 = out2;
  p.shift = shift; p.state = state; p.state_stride = state_stride;
  p.row_seq = row_seq; p.seq_q_start = seq_q_start; p.seq_q_len = seq_q_len; p.seq_state_slot = seq_state_slot;
  p.rows = rows; p.n = n; p.D = D;
  return p;
}
KVCM_API int kvcm_norm_pair_f32(KVCM_NORM_PAIR_ARGS) {
  return launch_norm_pair<float>(norm_pair_params(x, x_out, p0, s0, p1, s1, p2, s2, ey, place, wt, top, w1, eps1, out1, w2, eps2, out2,
                                                  shift, state, state_stride, row_seq, seq_q_start, seq_q_len, seq_state_slot, rows,
                                                  n, D, stream), (cudaStream_t)stream);
}
KVCM_API int kvcm_norm_pair_bf16(KVCM_NORM_PAIR_ARGS) {
  return launch_norm_pair<bf16>(norm_pair_params(x, x_out, p0, s0, p1, s1, p2, s2, ey, place, wt, top, w1, eps1, out1, w2, eps2, out2,
                                                 shift, state, state_stride, row_seq, seq_q_start, seq_q_len, seq_state_slot, rows,
                                                 n, D, stream), (cudaStream_t)stream);
}
