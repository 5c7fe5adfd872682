// The linear recurrence with ONE constant decay per head over the portions of a step, in chunks on tensor cores:
//
//     S <- d S + k v^T;   o = S^T q            per head, S [dk, dv] float, from and into the request's state row
//
// The token-by-token kernel (delta_rule.cu) is one dependent chain as long as the portion.  With a constant decay the chain
// can be cut: for the n tokens of a chunk that starts with state S,
//
//     o_i = d^(i+1) S^T q_i + sum_{j <= i} d^(i-j) (q_i . k_j) v_j
//     S'  = d^n S + P,   P = sum_j d^(n-1-j) k_j v_j^T
//
// so three launches serve every chunk (the batch's tiles of 64 rows) of every request at once:
//   1. outer : P of every (chunk, head)                                     tensor cores, all chunks side by side
//   2. carry : per request and element of S, S' along the request's chunks; P's place takes the S a chunk starts with
//   3. read  : o of every (chunk, head)                                     tensor cores, all chunks side by side
// No power of the decay is ever divided by: every factor is d^m with m >= 0.
//
// Precision: q, k and v (after the optional SiLU) are bfloat16 operands, as the projections of a 16-bit model may be.
// Whatever belongs to the recurrence is kept to more than float's 16 leading bits: operands that hold a decay or the state
// (d^m k, S, the decayed scores) are split into two bfloat16 parts, x = hi + lo with |x - hi - lo| <= 2^-17 |x|, and
// multiplied in two products; all sums, P and S are float.
// (Portions of one token, float storage and key sizes beyond 128 stay with the token-by-token kernel.)
#include "attention_mma.cuh"
#include "pdl.cuh"

namespace kvcm {

constexpr int kLcRows = 64;                // tokens of a chunk (the batch builder's tile)
constexpr int kLcCols = 64;                // columns of S per block
constexpr int kLcThreads = 128;

struct LinearChunkParams {
  const float* proj; int ld; int q_base, k_base, v_base;
  const float* decay;                      // [heads]
  float* carry;                            // [tiles, heads, dk, dv]
  float* state; long long state_stride;
  const int* tile_seq; const int* tile_q0; const int* seq_q_start; const int* seq_q_len; const int* seq_state_slot;
  float* out;                              // [rows, heads * dv]
  int tiles, heads, qk_heads, dk, dv, silu, vec;
};

__device__ __forceinline__ float lc_act(float z, int silu) { return silu ? z / (1.f + expf(-z)) : z; }

// hi + lo = x up to 2^-17 |x|
__device__ __forceinline__ void lc_split(float x, bf16& hi, bf16& lo) {
  hi = __float2bfloat16_rn(x);
  lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}

// Rows [0, kLcRows) of W neighbouring columns of the projection (activated, zero beyond n rows and `width` columns), each
// handed to `put(row, column, value)`; 16-byte loads where they are aligned.
template <int W, typename Put>
__device__ __forceinline__ void lc_rows(const float* src, int ld, int n, int width, int silu, int vec, Put put) {
  if (vec) {
    for (int i = threadIdx.x; i < kLcRows * (W / 4); i += kLcThreads) {
      const int r = i / (W / 4), c = (i - r * (W / 4)) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (r < n && c < width) v = *reinterpret_cast<const float4*>(src + size_t(r) * ld + c);      // (width % 4 == 0)
      put(r, c, lc_act(v.x, silu)); put(r, c + 1, lc_act(v.y, silu)); put(r, c + 2, lc_act(v.z, silu)); put(r, c + 3, lc_act(v.w, silu));
    }
  } else {
    for (int i = threadIdx.x; i < kLcRows * W; i += kLcThreads) {
      const int r = i / W, c = i - r * W;
      put(r, c, r < n && c < width ? lc_act(src[size_t(r) * ld + c], silu) : 0.f);
    }
  }
}

// A fragment (16 x 16) of the transpose of a tile stored [k][m]: the four 8 x 8 matrices transposed as they are loaded.
__device__ __forceinline__ void lc_frag_trans(uint32_t (&a)[4], const bf16* tile, int ldm, int lane) {
  const int mi = lane >> 3;
  ldmatrix_x4_trans(a, tile + ((mi >> 1) * 8 + (lane & 7)) * ldm + (mi & 1) * 8);
}

template <int DK>
__global__ void __launch_bounds__(kLcThreads)
linear_chunk_outer_kernel(LinearChunkParams p) {
  constexpr int LDK = DK + 8, LDV = kLcCols + 8;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* khi = reinterpret_cast<bf16*>(smem_raw);             // [64][LDK] d^(n-1-j) k_j
  bf16* klo = khi + kLcRows * LDK;
  bf16* vs = klo + kLcRows * LDK;                             // [64][LDV]
  __shared__ float pw[kLcRows + 1];
  pdl_launch_dependents();
  const int tile = blockIdx.x, head = blockIdx.y, c0 = blockIdx.z * kLcCols;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = p.tile_seq[tile], q0 = p.tile_q0[tile];
  const int row0 = p.seq_q_start[seq] + q0, n = min(kLcRows, p.seq_q_len[seq] - q0);
  const float d = p.decay[head];
  if (tid <= kLcRows) pw[tid] = powf(d, float(tid));
  __syncthreads();
  pdl_wait();
  const float* src = p.proj + size_t(row0) * p.ld;
  lc_rows<DK>(src + p.k_base + (head / (p.heads / p.qk_heads)) * p.dk, p.ld, n, p.dk, p.silu, p.vec, [&](int r, int c, float x) {
    // the key as a bfloat16 operand, then times its power of the decay in two parts
    lc_split(__bfloat162float(__float2bfloat16_rn(x)) * (r < n ? pw[n - 1 - r] : 0.f), khi[r * LDK + c], klo[r * LDK + c]);
  });
  lc_rows<kLcCols>(src + p.v_base + head * p.dv + c0, p.ld, n, p.dv - c0, p.silu, p.vec,
                   [&](int r, int c, float x) { vs[r * LDV + c] = __float2bfloat16_rn(x); });
  __syncthreads();
  float* dst = p.carry + (size_t(tile) * p.heads + head) * p.dk * p.dv;
  const int g = lane >> 2, t4 = lane & 3;
  for (int mt = warp; mt < DK / 16; mt += kLcThreads / 32) {
    if (mt * 16 >= p.dk) break;
    float o[kLcCols / 8][4];
#pragma unroll
    for (int i = 0; i < kLcCols / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < kLcRows / 16; ++kk) {
      uint32_t a[4];
      lc_frag_trans(a, khi + kk * 16 * LDK + mt * 16, LDK, lane);
      pv_16x16<kLcCols>(o, a, vs + kk * 16 * LDV, lane);
      lc_frag_trans(a, klo + kk * 16 * LDK + mt * 16, LDK, lane);
      pv_16x16<kLcCols>(o, a, vs + kk * 16 * LDV, lane);
    }
#pragma unroll
    for (int i = 0; i < kLcCols / 8; ++i)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int r = mt * 16 + g + 8 * h, c = c0 + 8 * i + 2 * t4;
        if (r >= p.dk) continue;
        float* at = dst + size_t(r) * p.dv + c;
        if ((p.dv & 1) == 0) {
          if (c < p.dv) *reinterpret_cast<float2*>(at) = make_float2(o[i][2 * h], o[i][2 * h + 1]);
        } else {
          if (c < p.dv) at[0] = o[i][2 * h];
          if (c + 1 < p.dv) at[1] = o[i][2 * h + 1];
        }
      }
  }
}

// One thread carries V neighbouring elements of one request's S along its chunks.
template <int V>
__global__ void __launch_bounds__(256)
linear_chunk_carry_kernel(LinearChunkParams p) {
  pdl_launch_dependents();
  const int tile0 = blockIdx.y;
  if (p.tile_q0[tile0] != 0) return;                          // a request's chunks belong to the block row of its first
  const int seq = p.tile_seq[tile0], len = p.seq_q_len[seq], slot = p.seq_state_slot[seq];
  const int per = p.dk * p.dv, total = p.heads * per;
  const int i = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (i >= total) return;
  const float d = p.decay[i / per];                           // (V divides a head's elements)
  const float whole = powf(d, float(kLcRows));
  pdl_wait();
  float S[V];
  float* st = slot >= 0 ? p.state + slot * p.state_stride + i : nullptr;
#pragma unroll
  for (int e = 0; e < V; ++e) S[e] = st ? st[e] : 0.f;
  float* at = p.carry + size_t(tile0) * total + i;
  const int n_tiles = (len + kLcRows - 1) / kLcRows;
  constexpr int AHEAD = 8;                                    // chunks whose P is asked for together
  for (int t0 = 0; t0 < n_tiles; t0 += AHEAD) {
    float P[AHEAD][V];
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
      if (t0 + j >= n_tiles) break;
      const float* src = at + size_t(t0 + j) * total;
      if constexpr (V == 4) {
        const float4 v = *reinterpret_cast<const float4*>(src);
        P[j][0] = v.x; P[j][1] = v.y; P[j][2] = v.z; P[j][3] = v.w;
      } else {
        P[j][0] = src[0];
      }
    }
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
      const int t = t0 + j;
      if (t >= n_tiles) break;
      float* dst = at + size_t(t) * total;
      if constexpr (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(S[0], S[1], S[2], S[3]);
      else dst[0] = S[0];
      const float f = t + 1 < n_tiles ? whole : powf(d, float(len - t * kLcRows));
#pragma unroll
      for (int e = 0; e < V; ++e) S[e] = fmaf(f, S[e], P[j][e]);
    }
  }
  if (st) {
#pragma unroll
    for (int e = 0; e < V; ++e) st[e] = S[e];
  }
}

template <int DK>
__global__ void __launch_bounds__(kLcThreads)
linear_chunk_read_kernel(LinearChunkParams p) {
  constexpr int LDK = DK + 8, LDV = kLcCols + 8;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* qs = reinterpret_cast<bf16*>(smem_raw);               // [64][LDK]
  bf16* ks = qs + kLcRows * LDK;                              // [64][LDK]
  bf16* vs = ks + kLcRows * LDK;                              // [64][LDV]
  bf16* shi = vs + kLcRows * LDV;                             // [DK][LDV]
  bf16* slo = shi + DK * LDV;
  __shared__ float pw[kLcRows + 1];
  pdl_launch_dependents();
  const int tile = blockIdx.x, head = blockIdx.y, c0 = blockIdx.z * kLcCols;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = p.tile_seq[tile], q0 = p.tile_q0[tile];
  const int row0 = p.seq_q_start[seq] + q0, n = min(kLcRows, p.seq_q_len[seq] - q0);
  if (tid <= kLcRows) pw[tid] = powf(p.decay[head], float(tid));
  pdl_wait();
  const float* src = p.proj + size_t(row0) * p.ld;
  const int qk = (head / (p.heads / p.qk_heads)) * p.dk;
  lc_rows<DK>(src + p.q_base + qk, p.ld, n, p.dk, p.silu, p.vec, [&](int r, int c, float x) { qs[r * LDK + c] = __float2bfloat16_rn(x); });
  lc_rows<DK>(src + p.k_base + qk, p.ld, n, p.dk, p.silu, p.vec, [&](int r, int c, float x) { ks[r * LDK + c] = __float2bfloat16_rn(x); });
  lc_rows<kLcCols>(src + p.v_base + head * p.dv + c0, p.ld, n, p.dv - c0, p.silu, p.vec,
                   [&](int r, int c, float x) { vs[r * LDV + c] = __float2bfloat16_rn(x); });
  const float* S = p.carry + (size_t(tile) * p.heads + head) * p.dk * p.dv + c0;
  const bool svec = p.vec != 0;                               // (dv % 4 == 0)
  for (int i = tid; i < DK * (kLcCols / 4); i += kLcThreads) {
    const int r = i / (kLcCols / 4), c = (i - r * (kLcCols / 4)) * 4;
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (r < p.dk) {
      if (svec) {
        if (c0 + c < p.dv) {
          const float4 a = *reinterpret_cast<const float4*>(S + size_t(r) * p.dv + c);
          v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
        }
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (c0 + c + e < p.dv) v[e] = S[size_t(r) * p.dv + c + e];
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) lc_split(v[e], shi[r * LDV + c + e], slo[r * LDV + c + e]);
  }
  __syncthreads();
  if (warp * 16 >= n) return;
  const int g = lane >> 2, t4 = lane & 3;
  uint32_t qa[DK / 16][4];
  load_q_frags<DK>(qa, qs + warp * 16 * LDK, lane);
  float o[kLcCols / 8][4];
#pragma unroll
  for (int i = 0; i < kLcCols / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
  for (int kk = 0; kk < DK / 16; ++kk) {
    pv_16x16<kLcCols>(o, qa[kk], shi + kk * 16 * LDV, lane);
    pv_16x16<kLcCols>(o, qa[kk], slo + kk * 16 * LDV, lane);
  }
  const int row[2] = {warp * 16 + g, warp * 16 + g + 8};      // this thread's rows of the chunk
#pragma unroll
  for (int i = 0; i < kLcCols / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[i][j] *= pw[row[j >> 1] + 1];
  for (int kb = 0; kb <= warp; ++kb) {                         // sixteen keys at a time, up to the rows' own
    float s[2][4];
    qk_16x16<DK>(s, qa, ks + kb * 16 * LDK, lane);
    float lo[2][4];
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int dist = row[j >> 1] - (kb * 16 + 8 * h + 2 * t4 + (j & 1));
        const float x = dist >= 0 ? s[h][j] * pw[dist] : 0.f;
        const float hi = __bfloat162float(__float2bfloat16_rn(x));
        s[h][j] = hi;
        lo[h][j] = x - hi;
      }
    const uint32_t ahi[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]), pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
    const uint32_t alo[4] = {pack_bf16(lo[0][0], lo[0][1]), pack_bf16(lo[0][2], lo[0][3]), pack_bf16(lo[1][0], lo[1][1]), pack_bf16(lo[1][2], lo[1][3])};
    pv_16x16<kLcCols>(o, ahi, vs + kb * 16 * LDV, lane);
    pv_16x16<kLcCols>(o, alo, vs + kb * 16 * LDV, lane);
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    if (row[h] >= n) continue;
    float* dst = p.out + size_t(row0 + row[h]) * p.heads * p.dv + size_t(head) * p.dv + c0 + 2 * t4;
#pragma unroll
    for (int i = 0; i < kLcCols / 8; ++i) {
      const int c = c0 + 8 * i + 2 * t4;
      if ((p.dv & 1) == 0) {
        if (c < p.dv) *reinterpret_cast<float2*>(dst + 8 * i) = make_float2(o[i][2 * h], o[i][2 * h + 1]);
      } else {
        if (c < p.dv) dst[8 * i] = o[i][2 * h];
        if (c + 1 < p.dv) dst[8 * i + 1] = o[i][2 * h + 1];
      }
    }
  }
}

template <int DK>
static int launch_linear_chunk(const LinearChunkParams& p, cudaStream_t s) {
  constexpr int LDK = DK + 8, LDV = kLcCols + 8;
  constexpr size_t smem_outer = size_t(2 * kLcRows * LDK + kLcRows * LDV) * sizeof(bf16);
  constexpr size_t smem_read = size_t(2 * kLcRows * LDK + kLcRows * LDV + 2 * DK * LDV) * sizeof(bf16);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(linear_chunk_outer_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem_outer));
    if (e == cudaSuccess) e = cudaFuncSetAttribute(linear_chunk_read_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem_read));
    if (e != cudaSuccess) return int(e);
    configured = true;
  }
  const dim3 grid(p.tiles, p.heads, (p.dv + kLcCols - 1) / kLcCols);
  int rc = pdl_launch(linear_chunk_outer_kernel<DK>, grid, dim3(kLcThreads), smem_outer, s, p);
  if (rc) return rc;
  const long long total = (long long)p.heads * p.dk * p.dv;
  if (((p.dk * p.dv) % 4) == 0 && (reinterpret_cast<uintptr_t>(p.carry) & 15) == 0)
    rc = pdl_launch(linear_chunk_carry_kernel<4>, dim3(unsigned((total / 4 + 255) / 256), p.tiles), dim3(256), 0, s, p);
  else
    rc = pdl_launch(linear_chunk_carry_kernel<1>, dim3(unsigned((total + 255) / 256), p.tiles), dim3(256), 0, s, p);
  if (rc) return rc;
  return pdl_launch(linear_chunk_read_kernel<DK>, grid, dim3(kLcThreads), smem_read, s, p);
}

}  // namespace kvcm

using namespace kvcm;

// Largest key size of the chunked form.
KVCM_API int kvcm_linear_chunk_max_dk(void) { return 128; }

// Runs the recurrence over the rows of every portion of more than one token (the step's tiles of 64 rows); single-row
// entries are not touched.  proj: float rows of `ld` elements with q, k, v at the given bases; decay [heads]; carry: float
// scratch [tiles, heads, dk, dv]; out: float [rows, heads * dv].
KVCM_API int kvcm_linear_chunk(const float* proj, int ld, int q_base, int k_base, int v_base, const float* decay, float* carry,
                               float* state, long long state_stride, const int* tile_seq, const int* tile_q0,
                               const int* seq_q_start, const int* seq_q_len, const int* seq_state_slot, float* out, int tiles,
                               int heads, int qk_heads, int dk, int dv, int silu, void* stream) {
  if (tiles == 0) return 0;
  if (dk < 1 || dk > 128 || dv < 1 || qk_heads < 1 || heads % qk_heads || tiles > 65535) return KVCM_ERR_UNSUPPORTED;
  LinearChunkParams p;
  p.proj = proj; p.ld = ld; p.q_base = q_base; p.k_base = k_base; p.v_base = v_base; p.decay = decay; p.carry = carry;
  p.state = state; p.state_stride = state_stride; p.tile_seq = tile_seq; p.tile_q0 = tile_q0; p.seq_q_start = seq_q_start;
  p.seq_q_len = seq_q_len; p.seq_state_slot = seq_state_slot; p.out = out; p.tiles = tiles; p.heads = heads;
  p.qk_heads = qk_heads; p.dk = dk; p.dv = dv; p.silu = silu;
  p.vec = (dk % 4) == 0 && (dv % 4) == 0 && (ld % 4) == 0 && (q_base % 4) == 0 && (k_base % 4) == 0 && (v_base % 4) == 0 &&
          ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(carry)) & 15) == 0;
  cudaStream_t s = (cudaStream_t)stream;
  if (dk <= 32) return launch_linear_chunk<32>(p, s);
  if (dk <= 64) return launch_linear_chunk<64>(p, s);
  return launch_linear_chunk<128>(p, s);
}
