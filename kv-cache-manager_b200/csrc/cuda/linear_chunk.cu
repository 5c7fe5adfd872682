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
//   1. outer : P of every (chunk, head)                                     tensor cores, all chunks side by side;
//              leaves the activated q, k and v as bfloat16 tiles for the third launch
//   2. carry : per request and element of S, S' along the request's chunks; leaves the S a chunk starts with, split
//   3. read  : o of every (chunk, head)                                     tensor cores, all chunks side by side
// What one launch leaves for the next lies in scratch as whole tiles (key sizes padded to 32, 64 or 128, value sizes to
// multiples of 64, missing rows and columns zero), so the third launch only copies.
// No power of the decay is ever divided by: every factor is d^m with m >= 0.
//
// Precision: q, k and v (after the optional SiLU) are bfloat16 operands, as the projections of a 16-bit model may be.
// Whatever belongs to the recurrence is kept to more than float's 16 leading bits: operands that hold a decay or the state
// (d^m k, S, the decayed scores) are split into two bfloat16 parts, x = hi + lo with |x - hi - lo| <= 2^-17 |x|, and
// multiplied in two products; all sums, P and S are float.  With `exact` the queries and keys are no plain projections
// (rotated, scaled) and are split the same way (products of two low parts, 2^-18 of a term, are left out).
// (Portions of one token, float storage and key sizes beyond 128 stay with the token-by-token kernel.)
#include "attention_mma.cuh"
#include "pdl.cuh"

namespace kvcm {

constexpr int kLcRows = 64;                // tokens of a chunk (the batch builder's tile)
constexpr int kLcCols = 64;                // columns of S per block
constexpr int kLcOuterThreads = 256, kLcReadThreads = 128;

struct LinearChunkParams {
  const float* proj; int ld; int q_base, k_base, v_base;
  const float* decay;                      // [heads]
  float* outer;                            // P      [tiles, heads, DK, DVP]
  bf16* split;                             // S      [tiles, heads, 2 (hi, lo), DK, DVP]
  bf16* q; bf16* k; bf16* v;               // [tiles, heads, 64, DK] twice, [tiles, heads, 64, DVP]
  bf16* q_lo; bf16* k_lo;                  // exact: the low parts of q and k, like them; else null
  float* state; long long state_stride;
  const int* tile_seq; const int* tile_q0; const int* seq_q_start; const int* seq_q_len; const int* seq_state_slot;
  float* out;                              // [rows, heads * dv]
  int tiles, heads, qk_heads, dk, dv, dvp, silu, vec;
  const float* cs; int half; float amplitude, k_scale;      // cs [rows][half cosines | half sines]: q and k turn in pairs (i, i + half); or null
};

__device__ __forceinline__ float lc_act(float z) { return z / (1.f + expf(-z)); }

// hi + lo = x up to 2^-17 |x|
__device__ __forceinline__ float lc_round(float x) { return __bfloat162float(__float2bfloat16_rn(x)); }

// Rows [0, kLcRows) of W neighbouring columns of the projection (activated, zero beyond n rows and `width` columns), four
// neighbouring values at a time handed to `put(row, column, values)`; 16-byte loads, eight of a thread in flight
// together, where they are aligned.
template <int W, typename Put>
__device__ __forceinline__ void lc_rows(const float* src, int ld, int n, int width, int silu, int vec, Put put) {
  constexpr int kQuads = kLcRows * (W / 4), kTurns = kQuads / kLcOuterThreads, kBatch = kTurns < 8 ? kTurns : 8;
  static_assert(kQuads % kLcOuterThreads == 0 && kTurns % kBatch == 0, "a thread's turns come in whole batches");
#pragma unroll 1
  for (int t = 0; t < kTurns; t += kBatch) {
    float v[kBatch][4];
#pragma unroll
    for (int b = 0; b < kBatch; ++b) {
      const int i = threadIdx.x + (t + b) * kLcOuterThreads, r = i / (W / 4), c = (i - r * (W / 4)) * 4;
      v[b][0] = v[b][1] = v[b][2] = v[b][3] = 0.f;
      if (r >= n) continue;
      const float* at = src + size_t(r) * ld + c;
      if (vec) {
        if (c < width) {                                       // (width % 4 == 0)
          const float4 f = *reinterpret_cast<const float4*>(at);
          v[b][0] = f.x; v[b][1] = f.y; v[b][2] = f.z; v[b][3] = f.w;
        }
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (c + e < width) v[b][e] = at[e];
      }
    }
#pragma unroll
    for (int b = 0; b < kBatch; ++b) {
      const int i = threadIdx.x + (t + b) * kLcOuterThreads, r = i / (W / 4), c = (i - r * (W / 4)) * 4;
      if (silu) {
#pragma unroll
        for (int e = 0; e < 4; ++e) v[b][e] = lc_act(v[b][e]);
      }
      put(r, c, v[b]);
    }
  }
}

// The same with the row's pairs (i, i + half), i < half, turned by the step's angles and everything multiplied by `scale`
// (vec, half % 4 == 0).  An item is four pairs or four elements behind them.
template <int W, typename Put>
__device__ __forceinline__ void lc_rows_turned(const LinearChunkParams& p, const float* src, int row0, int n, float scale, Put put) {
  const int pairs = p.half / 4, per = W / 4 - pairs, total = kLcRows * per;
  constexpr int kBatch = 4;
#pragma unroll 1
  for (int i0 = threadIdx.x; i0 < total; i0 += kBatch * kLcOuterThreads) {
    float a[kBatch][4], b[kBatch][4], c[kBatch][4], s[kBatch][4];
#pragma unroll
    for (int t = 0; t < kBatch; ++t) {
      const int i = i0 + t * kLcOuterThreads, r = i / per, k = i - r * per;
      const bool turn = k < pairs;
      const int at = turn ? 4 * k : 2 * p.half + 4 * (k - pairs);
#pragma unroll
      for (int e = 0; e < 4; ++e) { a[t][e] = b[t][e] = s[t][e] = 0.f; c[t][e] = 1.f; }
      if (i >= total || r >= n || at >= p.dk) continue;
      const float4 f = *reinterpret_cast<const float4*>(src + size_t(r) * p.ld + at);
      a[t][0] = f.x; a[t][1] = f.y; a[t][2] = f.z; a[t][3] = f.w;
      if (turn) {
        const float4 g = *reinterpret_cast<const float4*>(src + size_t(r) * p.ld + at + p.half);
        const float* cs = p.cs + size_t(row0 + r) * 2 * p.half + at;
        const float4 co = *reinterpret_cast<const float4*>(cs), si = *reinterpret_cast<const float4*>(cs + p.half);
        b[t][0] = g.x; b[t][1] = g.y; b[t][2] = g.z; b[t][3] = g.w;
        c[t][0] = co.x; c[t][1] = co.y; c[t][2] = co.z; c[t][3] = co.w;
        s[t][0] = si.x; s[t][1] = si.y; s[t][2] = si.z; s[t][3] = si.w;
      }
    }
#pragma unroll
    for (int t = 0; t < kBatch; ++t) {
      const int i = i0 + t * kLcOuterThreads, r = i / per, k = i - r * per;
      if (i >= total) break;
      const bool turn = k < pairs;
      const int at = turn ? 4 * k : 2 * p.half + 4 * (k - pairs);
      float x[4], y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (turn) rotate_pair(a[t][e], b[t][e], c[t][e] * p.amplitude, s[t][e] * p.amplitude, x[e], y[e]);
        else x[e] = a[t][e];
        x[e] *= scale;
        y[e] *= scale;
      }
      put(r, at, x);
      if (turn) put(r, at + p.half, y);
    }
  }
}

// Four neighbouring bfloat16 values as one 8-byte store (tile rows are an even number of elements wide).
__device__ __forceinline__ void lc_store4(bf16* dst, float a, float b, float c, float d) {
  uint2 raw;
  raw.x = pack_bf16(a, b);
  raw.y = pack_bf16(c, d);
  *reinterpret_cast<uint2*>(dst) = raw;
}

// A fragment (16 x 16) of the transpose of a tile stored [k][m]: the four 8 x 8 matrices transposed as they are loaded.
__device__ __forceinline__ void lc_frag_trans(uint32_t (&a)[4], const bf16* tile, int ldm, int lane) {
  const int mi = lane >> 3;
  ldmatrix_x4_trans(a, tile + ((mi >> 1) * 8 + (lane & 7)) * ldm + (mi & 1) * 8);
}

// O (16 x 64) += A (16 x 16) * B (16 x 64), B stored [k][column] at a row stride of ldv.
__device__ __forceinline__ void lc_pv_64(float (&o)[8][4], const uint32_t (&a)[4], const bf16* tile, int ldv, int lane) {
  const int row = (lane & 7) + (((lane >> 3) & 1) << 3), col = (lane >> 4) << 3;
#pragma unroll
  for (int dd = 0; dd < 4; ++dd) {
    uint32_t b[4];
    ldmatrix_x4_trans(b, tile + row * ldv + dd * 16 + col);
    mma_bf16(o[2 * dd], a, b[0], b[1]);
    mma_bf16(o[2 * dd + 1], a, b[2], b[3]);
  }
}

template <int DK, int DVB, bool TURN>          // DVB: columns of S a block forms; TURN: q and k are turned and scaled on their way in
__global__ void __launch_bounds__(kLcOuterThreads, 2)
linear_chunk_outer_kernel(LinearChunkParams p) {
  constexpr int LDK = DK + 8, LDV = DVB + 8;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* khi = reinterpret_cast<bf16*>(smem_raw);             // [64][LDK] d^(n-1-j) k_j
  bf16* klo = khi + kLcRows * LDK;
  bf16* vs = klo + kLcRows * LDK;                             // [64][LDV]
  __shared__ float pw[kLcRows + 1];
  pdl_launch_dependents();
  const int tile = blockIdx.x, head = blockIdx.y, c0 = blockIdx.z * DVB;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = p.tile_seq[tile], q0 = p.tile_q0[tile];
  const int row0 = p.seq_q_start[seq] + q0, n = min(kLcRows, p.seq_q_len[seq] - q0);
  if (tid <= kLcRows) pw[tid] = powf(p.decay[head], float(tid));
  __syncthreads();
  pdl_wait();
  const float* src = p.proj + size_t(row0) * p.ld;
  const int qk = (head / (p.heads / p.qk_heads)) * p.dk;
  const size_t th = size_t(tile) * p.heads + head;
  const bool first = blockIdx.z == 0;                         // leaves q and k too
  bf16* qg = p.q + th * kLcRows * DK;
  bf16* kg = p.k + th * kLcRows * DK;
  bf16* vg = p.v + th * kLcRows * p.dvp + c0;
  auto put_k = [&](int r, int c, const float (&x)[4]) {
    // the key as a bfloat16 operand, then times its power of the decay in two parts
    const float f = r < n ? pw[n - 1 - r] : 0.f;
    float y[4], hi[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      y[e] = (p.k_lo ? x[e] : lc_round(x[e])) * f;
      hi[e] = lc_round(y[e]);
    }
    lc_store4(khi + r * LDK + c, hi[0], hi[1], hi[2], hi[3]);
    lc_store4(klo + r * LDK + c, y[0] - hi[0], y[1] - hi[1], y[2] - hi[2], y[3] - hi[3]);
    if (first) {
      lc_store4(kg + r * DK + c, x[0], x[1], x[2], x[3]);
      if (p.k_lo) lc_store4(p.k_lo + th * kLcRows * DK + r * DK + c, x[0] - lc_round(x[0]), x[1] - lc_round(x[1]), x[2] - lc_round(x[2]), x[3] - lc_round(x[3]));
    }
  };
  if constexpr (TURN) lc_rows_turned<DK>(p, src + p.k_base + qk, row0, n, p.k_scale, put_k);
  else lc_rows<DK>(src + p.k_base + qk, p.ld, n, p.dk, p.silu, p.vec, put_k);
  lc_rows<DVB>(src + p.v_base + head * p.dv + c0, p.ld, n, p.dv - c0, p.silu, p.vec, [&](int r, int c, const float (&x)[4]) {
    lc_store4(vs + r * LDV + c, x[0], x[1], x[2], x[3]);
    lc_store4(vg + r * p.dvp + c, x[0], x[1], x[2], x[3]);
  });
  if (first) {
    auto put_q = [&](int r, int c, const float (&x)[4]) {
      lc_store4(qg + r * DK + c, x[0], x[1], x[2], x[3]);
      if (p.q_lo) lc_store4(p.q_lo + th * kLcRows * DK + r * DK + c, x[0] - lc_round(x[0]), x[1] - lc_round(x[1]), x[2] - lc_round(x[2]), x[3] - lc_round(x[3]));
    };
    if constexpr (TURN) lc_rows_turned<DK>(p, src + p.q_base + qk, row0, n, 1.f, put_q);
    else lc_rows<DK>(src + p.q_base + qk, p.ld, n, p.dk, p.silu, p.vec, put_q);
  }
  __syncthreads();
  float* dst = p.outer + th * DK * p.dvp + c0;
  const int g = lane >> 2, t4 = lane & 3;
  for (int task = warp; task < (DK / 16) * (DVB / 64); task += kLcOuterThreads / 32) {       // 16 rows x 64 columns of P
    const int mt = task % (DK / 16), nb = task / (DK / 16) * 64;
    float o[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < kLcRows / 16; ++kk) {
      uint32_t a[4], b[4];
      lc_frag_trans(a, khi + kk * 16 * LDK + mt * 16, LDK, lane);
      lc_frag_trans(b, klo + kk * 16 * LDK + mt * 16, LDK, lane);
      lc_pv_64(o, a, vs + kk * 16 * LDV + nb, LDV, lane);
      lc_pv_64(o, b, vs + kk * 16 * LDV + nb, LDV, lane);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int h = 0; h < 2; ++h)
        *reinterpret_cast<float2*>(dst + size_t(mt * 16 + g + 8 * h) * p.dvp + nb + 8 * i + 2 * t4) = make_float2(o[i][2 * h], o[i][2 * h + 1]);
  }
}

// One thread carries four neighbouring elements of one request's (padded) S along its chunks.
__global__ void __launch_bounds__(256)
linear_chunk_carry_kernel(LinearChunkParams p, int DK) {
  pdl_launch_dependents();
  const int tile0 = blockIdx.y;
  if (p.tile_q0[tile0] != 0) return;                          // a request's chunks belong to the block row of its first
  const int seq = p.tile_seq[tile0], len = p.seq_q_len[seq], slot = p.seq_state_slot[seq];
  const int per = DK * p.dvp, total = p.heads * per;          // (dvp is a multiple of 64)
  const int i = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (i >= total) return;
  const int head = i / per, in = i - head * per, r = in / p.dvp, c = in - r * p.dvp;
  const float d = p.decay[head];
  const float whole = powf(d, float(kLcRows));
  const int n_tiles = (len + kLcRows - 1) / kLcRows;
  const float last = powf(d, float(len - (n_tiles - 1) * kLcRows));
  const int live = r < p.dk ? min(4, p.dv - c) : 0;           // elements that the state holds
  float* st = slot >= 0 ? p.state + slot * p.state_stride + (size_t(head) * p.dk + r) * p.dv + c : nullptr;
  pdl_wait();
  float S[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int e = 0; e < 4; ++e)
    if (st && e < live) S[e] = st[e];
  const float* src = p.outer + size_t(tile0) * total + i;
  bf16* dst = p.split + 2 * (size_t(tile0) * total + size_t(head) * per) + in;
  constexpr int AHEAD = 8;                                    // chunks whose P is asked for together
  for (int t0 = 0; t0 < n_tiles; t0 += AHEAD) {
    float4 P[AHEAD];
#pragma unroll
    for (int j = 0; j < AHEAD; ++j)
      if (t0 + j < n_tiles) P[j] = *reinterpret_cast<const float4*>(src + size_t(t0 + j) * total);
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
      const int t = t0 + j;
      if (t >= n_tiles) break;
      float hi[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) hi[e] = lc_round(S[e]);
      bf16* at = dst + 2 * size_t(t) * total;
      lc_store4(at, hi[0], hi[1], hi[2], hi[3]);
      lc_store4(at + per, S[0] - hi[0], S[1] - hi[1], S[2] - hi[2], S[3] - hi[3]);
      const float f = t + 1 < n_tiles ? whole : last;
      S[0] = fmaf(f, S[0], P[j].x); S[1] = fmaf(f, S[1], P[j].y); S[2] = fmaf(f, S[2], P[j].z); S[3] = fmaf(f, S[3], P[j].w);
    }
  }
#pragma unroll
  for (int e = 0; e < 4; ++e)
    if (st && e < live) st[e] = S[e];
}

// Copies a [rows][W] bfloat16 tile (row stride lds elements in memory) to shared memory rows of W + 8 elements.
template <int W>
__device__ __forceinline__ void lc_copy_tile(bf16* dst, const bf16* src, int rows, int lds) {
  constexpr int CH = W / 8;
  for (int i = threadIdx.x; i < rows * CH; i += kLcReadThreads) {
    const int r = i / CH, c = (i - r * CH) * 8;
    cp_async16(dst + r * (W + 8) + c, src + size_t(r) * lds + c);
  }
}

// EXACT: q and k in two parts each; the low part of q waits behind S, that of k takes the place of q once q is in registers.
template <int DK, bool EXACT>
__global__ void __launch_bounds__(kLcReadThreads)
linear_chunk_read_kernel(LinearChunkParams p) {
  constexpr int LDK = DK + 8, LDV = kLcCols + 8;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* qs = reinterpret_cast<bf16*>(smem_raw);               // [64][LDK]
  bf16* ks = qs + kLcRows * LDK;                              // [64][LDK]
  bf16* vs = ks + kLcRows * LDK;                              // [64][LDV]
  bf16* shi = vs + kLcRows * LDV;                             // [DK][LDV]
  bf16* slo = shi + DK * LDV;
  bf16* qls = slo + DK * LDV;                                 // EXACT: [64][LDK]
  __shared__ float pw[kLcRows + 1];
  pdl_launch_dependents();
  const int tile = blockIdx.x, head = blockIdx.y, c0 = blockIdx.z * kLcCols;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = p.tile_seq[tile], q0 = p.tile_q0[tile];
  const int row0 = p.seq_q_start[seq] + q0, n = min(kLcRows, p.seq_q_len[seq] - q0);
  if (tid <= kLcRows) pw[tid] = powf(p.decay[head], float(tid));
  pdl_wait();
  const size_t th = size_t(tile) * p.heads + head;
  const bf16* S = p.split + 2 * th * DK * p.dvp + c0;
  lc_copy_tile<DK>(qs, p.q + th * kLcRows * DK, kLcRows, DK);
  if constexpr (EXACT) lc_copy_tile<DK>(qls, p.q_lo + th * kLcRows * DK, kLcRows, DK);
  lc_copy_tile<kLcCols>(shi, S, DK, p.dvp);
  lc_copy_tile<kLcCols>(slo, S + size_t(DK) * p.dvp, DK, p.dvp);
  cp_async_commit();
  lc_copy_tile<DK>(ks, p.k + th * kLcRows * DK, kLcRows, DK);
  lc_copy_tile<kLcCols>(vs, p.v + th * kLcRows * p.dvp + c0, kLcRows, p.dvp);
  cp_async_commit();
  cp_async_wait<1>();
  __syncthreads();
  const int g = lane >> 2, t4 = lane & 3;
  uint32_t qa[DK / 16][4];
  load_q_frags<DK>(qa, qs + warp * 16 * LDK, lane);
  uint32_t ql[EXACT ? DK / 16 : 1][4];
  if constexpr (EXACT) {
    load_q_frags<DK>(reinterpret_cast<uint32_t(&)[DK / 16][4]>(ql), qls + warp * 16 * LDK, lane);
    __syncthreads();                                           // every warp has its rows of q
    lc_copy_tile<DK>(qs, p.k_lo + th * kLcRows * DK, kLcRows, DK);
    cp_async_commit();
  }
  float o[kLcCols / 8][4];
#pragma unroll
  for (int i = 0; i < kLcCols / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
  for (int kk = 0; kk < DK / 16; ++kk) {
    pv_16x16<kLcCols>(o, qa[kk], shi + kk * 16 * LDV, lane);
    pv_16x16<kLcCols>(o, qa[kk], slo + kk * 16 * LDV, lane);
    if constexpr (EXACT) pv_16x16<kLcCols>(o, ql[kk], shi + kk * 16 * LDV, lane);
  }
  cp_async_wait<0>();
  __syncthreads();                                             // every thread's share of k and v is there
  if (warp * 16 >= n) return;
  const int row[2] = {warp * 16 + g, warp * 16 + g + 8};      // this thread's rows of the chunk
#pragma unroll
  for (int i = 0; i < kLcCols / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[i][j] *= pw[row[j >> 1] + 1];
  for (int kb = 0; kb <= warp; ++kb) {                         // sixteen keys at a time, up to the rows' own
    float s[2][4];
    qk_16x16<DK>(s, qa, ks + kb * 16 * LDK, lane);
    if constexpr (EXACT) {
      float a[2][4], b[2][4];
      qk_16x16<DK>(a, reinterpret_cast<const uint32_t(&)[DK / 16][4]>(ql), ks + kb * 16 * LDK, lane);
      qk_16x16<DK>(b, qa, qs + kb * 16 * LDK, lane);
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int j = 0; j < 4; ++j) s[h][j] += a[h][j] + b[h][j];
    }
    float lo[2][4];
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int dist = row[j >> 1] - (kb * 16 + 8 * h + 2 * t4 + (j & 1));
        const float x = dist >= 0 ? s[h][j] * pw[dist] : 0.f;
        const float hi = lc_round(x);
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

// Scratch of a launch, in bytes from a 16-byte aligned start: P, then S split, q, k, v (every part a multiple of 16).
struct LinearChunkScratch { long long outer, split, q, k, v, q_lo, k_lo, total; };
static LinearChunkScratch linear_chunk_scratch(int tiles, int heads, int DK, int dvp, int exact) {
  const long long th = (long long)tiles * heads;
  LinearChunkScratch s;
  s.outer = 0;
  s.split = s.outer + th * DK * dvp * 4;
  s.q = s.split + th * DK * dvp * 4;
  s.k = s.q + th * kLcRows * DK * 2;
  s.v = s.k + th * kLcRows * DK * 2;
  s.q_lo = s.v + th * kLcRows * dvp * 2;
  s.k_lo = s.q_lo + (exact ? th * kLcRows * DK * 2 : 0);
  s.total = s.k_lo + (exact ? th * kLcRows * DK * 2 : 0);
  return s;
}
static int linear_chunk_dk(int dk) { return dk <= 32 ? 32 : dk <= 64 ? 64 : 128; }
static int linear_chunk_dvp(int dv) { return (dv + 63) / 64 * 64; }

template <int DK, int DVB, bool TURN>
static int launch_linear_outer_as(const LinearChunkParams& p, cudaStream_t s) {
  constexpr size_t smem = size_t(2 * kLcRows * (DK + 8) + kLcRows * (DVB + 8)) * sizeof(bf16);
  static bool configured = false;
  if (!configured && smem > 40 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(linear_chunk_outer_kernel<DK, DVB, TURN>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    if (e != cudaSuccess) return int(e);
    configured = true;
  }
  return pdl_launch(linear_chunk_outer_kernel<DK, DVB, TURN>, dim3(p.tiles, p.heads, p.dvp / DVB), dim3(kLcOuterThreads), smem, s, p);
}
template <int DK, int DVB>
static int launch_linear_outer(const LinearChunkParams& p, cudaStream_t s) {
  return p.cs ? launch_linear_outer_as<DK, DVB, true>(p, s) : launch_linear_outer_as<DK, DVB, false>(p, s);
}

template <int DK, bool EXACT>
static int launch_linear_chunk_as(const LinearChunkParams& p, cudaStream_t s) {
  constexpr size_t smem = size_t((EXACT ? 3 : 2) * kLcRows * (DK + 8) + kLcRows * (kLcCols + 8) + 2 * DK * (kLcCols + 8)) * sizeof(bf16);
  static bool configured = false;
  if (!configured && smem > 40 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(linear_chunk_read_kernel<DK, EXACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    if (e != cudaSuccess) return int(e);
    configured = true;
  }
  int rc = (p.dvp % 128) == 0 ? launch_linear_outer<DK, 128>(p, s) : launch_linear_outer<DK, 64>(p, s);
  if (rc) return rc;
  const long long quads = (long long)p.heads * DK * p.dvp / 4;
  rc = pdl_launch(linear_chunk_carry_kernel, dim3(unsigned((quads + 255) / 256), p.tiles), dim3(256), 0, s, p, DK);
  if (rc) return rc;
  return pdl_launch(linear_chunk_read_kernel<DK, EXACT>, dim3(p.tiles, p.heads, p.dvp / kLcCols), dim3(kLcReadThreads), smem, s, p);
}
template <int DK>
static int launch_linear_chunk(const LinearChunkParams& p, cudaStream_t s) {
  return p.q_lo ? launch_linear_chunk_as<DK, true>(p, s) : launch_linear_chunk_as<DK, false>(p, s);
}

}  // namespace kvcm

using namespace kvcm;

// Largest key size of the chunked form.
KVCM_API int kvcm_linear_chunk_max_dk(void) { return 128; }

// Bytes of scratch for a step of `tiles` chunks.
KVCM_API long long kvcm_linear_chunk_scratch_bytes(int tiles, int heads, int dk, int dv, int exact) {
  return linear_chunk_scratch(tiles, heads, linear_chunk_dk(dk), linear_chunk_dvp(dv), exact).total;
}

// Runs the recurrence over the rows of every portion of more than one token (the step's tiles of 64 rows); single-row
// entries are not touched.  proj: float rows of `ld` elements with q, k, v at the given bases; decay [heads]; scratch:
// kvcm_linear_chunk_scratch_bytes(), 16-byte aligned; cs (optional): q and k are turned on their way in, k times k_scale; out: float [rows, heads * dv].
KVCM_API int kvcm_linear_chunk(const float* proj, int ld, int q_base, int k_base, int v_base, const float* decay, void* scratch,
                               float* state, long long state_stride, const int* tile_seq, const int* tile_q0,
                               const int* seq_q_start, const int* seq_q_len, const int* seq_state_slot, float* out, int tiles,
                               int heads, int qk_heads, int dk, int dv, int silu, int exact, const float* cs, int half, float amplitude,
                               float k_scale, void* stream) {
  if (tiles == 0) return 0;
  if (dk < 1 || dk > 128 || dv < 1 || qk_heads < 1 || heads % qk_heads || tiles > 65535 || heads > 65535 ||
      (reinterpret_cast<uintptr_t>(scratch) & 15))
    return KVCM_ERR_UNSUPPORTED;
  LinearChunkParams p;
  p.proj = proj; p.ld = ld; p.q_base = q_base; p.k_base = k_base; p.v_base = v_base; p.decay = decay;
  p.state = state; p.state_stride = state_stride; p.tile_seq = tile_seq; p.tile_q0 = tile_q0; p.seq_q_start = seq_q_start;
  p.seq_q_len = seq_q_len; p.seq_state_slot = seq_state_slot; p.out = out; p.tiles = tiles; p.heads = heads;
  p.qk_heads = qk_heads; p.dk = dk; p.dv = dv; p.dvp = linear_chunk_dvp(dv); p.silu = silu;
  const LinearChunkScratch at = linear_chunk_scratch(tiles, heads, linear_chunk_dk(dk), p.dvp, exact);
  char* base = static_cast<char*>(scratch);
  p.outer = reinterpret_cast<float*>(base + at.outer); p.split = reinterpret_cast<bf16*>(base + at.split);
  p.q = reinterpret_cast<bf16*>(base + at.q); p.k = reinterpret_cast<bf16*>(base + at.k); p.v = reinterpret_cast<bf16*>(base + at.v);
  p.q_lo = exact ? reinterpret_cast<bf16*>(base + at.q_lo) : nullptr; p.k_lo = exact ? reinterpret_cast<bf16*>(base + at.k_lo) : nullptr;
  p.vec = (dk % 4) == 0 && (dv % 4) == 0 && (ld % 4) == 0 && (q_base % 4) == 0 && (k_base % 4) == 0 && (v_base % 4) == 0 &&
          (reinterpret_cast<uintptr_t>(proj) & 15) == 0;
  p.cs = cs; p.half = half; p.amplitude = amplitude; p.k_scale = k_scale;
  if (cs && (!p.vec || silu || half < 4 || half % 4 || 2 * half > dk || (reinterpret_cast<uintptr_t>(cs) & 15))) return KVCM_ERR_UNSUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
  if (dk <= 32) return launch_linear_chunk<32>(p, s);
  if (dk <= 64) return launch_linear_chunk<64>(p, s);
  return launch_linear_chunk<128>(p, s);
}
