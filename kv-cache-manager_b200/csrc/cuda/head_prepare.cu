// From a float projection of a step's rows to what the kernels behind it read, head by head, for up to kMaxHeadSegments
// runs of equal heads ("segments") of one row layout in ONE launch.  A segment's heads
//
//   1. optionally pass a short causal convolution over time, channel by channel (no bias, no activation):
//        y_t = sum_j w[channel, j] u_(t - taps + 1 + j),   u before the portion from the request's state row
//   2. optionally turn their first 2 * half dimensions by position * inv_freq (table 0 or 1), in rotate-half pairs
//      (i, i + half) or interleaved ones (2i, 2i + 1); cosines and sines times the table's amplitude
//   3. are multiplied by `scale`
//   4. go to rows of padded heads in the storage type (zeros beyond a head's own size), to the row's page slot
//      [pages, heads, page, HD] in the storage type, or to float rows (in place where the segment has no convolution)
//
// The convolved channels are `channels` neighbouring columns of the projection from `conv_col` on; a request's state row keeps
// the last taps - 1 of them ([taps - 1][channels] floats, the oldest first; zeros at its start).  In a step whose requests
// all bring one row each the same launch moves the state on; otherwise a second small launch does, behind this one.
//
// There is no reduction anywhere: a work item is four neighbouring elements of a head (in rotate-half pairs, two times
// four), for R rows of the step at a time, whose inputs are each read once.  Sizes that are not multiples of four, more
// than four taps and unaligned rows take an element-wise kernel.  Everything is float.
#include "common.cuh"
#include "pdl.cuh"

namespace kvcm {

constexpr int kMaxHeadSegments = 6;
constexpr int kHeadPrepareThreads = 256;
constexpr int kHeadRunRows = 4;
enum HeadDest { kHeadRows = 0, kHeadPages = 1, kHeadFloatRows = 2 };

struct HeadSegment {                       // (mirrored by kernels/library.py)
  void* out; long long ld;                 // rows: elements from one row to the next
  int units, dim, HD;                      // heads, elements of a head, of a padded head (float rows: HD == dim)
  int src, conv;                           // first column of the projection; first convolved channel or -1
  int table, interleaved, dest;            // rotation table or -1
  float scale;
  int rows;                                // rows of the step that the segment covers, from the first on
  int items;                               // work items of a head (filled in by the launcher)
};
struct HeadPrepareParams {
  const float* proj; long long ldp;
  const int* positions;
  const float* inv_freq[2]; const float* cs[2]; int half[2]; float amplitude[2];      // cs: [rows][half cosines | half sines] (used for many rows) or null
  const float* conv_w; float* state; long long state_stride;
  int taps, channels, conv_col, write_state;
  const int* row_seq; const int* seq_q_start; const int* seq_q_len; const int* seq_state_slot;
  const int* slot_mapping; int block_size;
  int rows, seqs, segments, items;
  HeadSegment seg[kMaxHeadSegments];
};

__device__ __forceinline__ void hp_store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void hp_store4(bf16* p, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  uint2 raw;
  raw.x = *reinterpret_cast<const uint32_t*>(&a);
  raw.y = *reinterpret_cast<const uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = raw;
}
__device__ __forceinline__ void hp_load4(float (&v)[4], const float* p) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}

// What a block's rows need besides the projection.
template <int R> struct HeadRowInfo {
  int local[R], state_slot[R], page[R], off[R];   // row of its portion, the request's state slot, the row's page (or -1) and place
  int whole;                                      // all rows are there and none reaches ahead of its portion
};

// Cosines and sines of R rows: [row][table 0: half cosines, half sines | table 1: ..], amplitude included
template <int R>
__device__ __forceinline__ void hp_tables(const HeadPrepareParams& p, int r0, float* cs) {
  const int n0 = p.half[0], n = n0 + p.half[1];
  for (int i = threadIdx.x; i < R * n; i += blockDim.x) {
    const int r = i / n, j = i - r * n;
    if (r0 + r >= p.rows) continue;
    const int t = j >= n0, k = t ? j - n0 : j;
    float sn, c;
    sincosf(float(p.positions[r0 + r]) * p.inv_freq[t][k], &sn, &c);
    float* at = cs + r * 2 * n + (t ? 2 * n0 : 0);
    at[k] = c * p.amplitude[t];
    at[p.half[t] + k] = sn * p.amplitude[t];
  }
}

// Four neighbouring elements (from element c of head u on) of R rows, convolved where the segment asks for it.
template <int TAPS, int R>
__device__ __forceinline__ void hp_quads(const HeadPrepareParams& p, const HeadSegment& g, const HeadRowInfo<R>& info, int r0, int u, int c,
                                         float (&v)[R][4]) {
  const int at = u * g.dim + c;
  const float* src = p.proj + g.src + at;
  if (TAPS == 1 || g.conv < 0) {
#pragma unroll
    for (int i = 0; i < R; ++i) {
      v[i][0] = v[i][1] = v[i][2] = v[i][3] = 0.f;
      if (r0 + i < p.rows) hp_load4(v[i], src + (r0 + i) * p.ldp);
    }
    if (TAPS == 1 && g.conv >= 0) {                  // a single tap: a factor per channel
      float w[4];
      hp_load4(w, p.conv_w + g.conv + at);
#pragma unroll
      for (int i = 0; i < R; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) v[i][e] *= w[e];
    }
    return;
  }
  if constexpr (TAPS > 1) {
  float raw[R + TAPS - 1][4], w[4 * TAPS];
  if (R > 1 && info.whole) {
    const float* from = src + (r0 - (TAPS - 1)) * p.ldp;
#pragma unroll
    for (int k = 0; k < R + TAPS - 1; ++k, from += p.ldp) hp_load4(raw[k], from);
  } else {
#pragma unroll
    for (int k = 0; k < R + TAPS - 1; ++k) {
      const int row = r0 + k - (TAPS - 1);
      raw[k][0] = raw[k][1] = raw[k][2] = raw[k][3] = 0.f;
      if (row >= 0 && row < p.rows) hp_load4(raw[k], src + row * p.ldp);
    }
  }
  const float* wp = p.conv_w + size_t(g.conv + at) * TAPS;
#pragma unroll
  for (int k = 0; k < TAPS; ++k) {
    float4 f = *reinterpret_cast<const float4*>(wp + 4 * k);
    w[4 * k] = f.x; w[4 * k + 1] = f.y; w[4 * k + 2] = f.z; w[4 * k + 3] = f.w;
  }
  if (R > 1 && info.whole) {
#pragma unroll
    for (int i = 0; i < R; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        v[i][e] = w[e * TAPS] * raw[i][e];
#pragma unroll
        for (int j = 1; j < TAPS; ++j) v[i][e] = fmaf(w[e * TAPS + j], raw[i + j][e], v[i][e]);
      }
    return;
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int local = info.local[i];
    float* kept = info.state_slot[i] >= 0 ? p.state + info.state_slot[i] * p.state_stride + g.conv + at : nullptr;
    v[i][0] = v[i][1] = v[i][2] = v[i][3] = 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int back = TAPS - 1 - j;
      float x[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) x[e] = raw[i + j][e];
      if (local < back) {                            // ahead of the portion: what earlier steps left
        x[0] = x[1] = x[2] = x[3] = 0.f;
        if (kept) hp_load4(x, kept + size_t(TAPS - 1 + local - back) * p.channels);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) v[i][e] = fmaf(w[e * TAPS + j], x[e], v[i][e]);
      // (single rows: tap j > 0 holds what the state's place j - 1 keeps from now on; this thread alone reads these channels)
      if (R == 1 && j > 0 && p.write_state && kept) hp_store4(kept + size_t(j - 1) * p.channels, x);
    }
  }
  }
}

template <typename T, int R>
__device__ __forceinline__ void hp_put(const HeadPrepareParams& p, const HeadSegment& g, const HeadRowInfo<R>& info, int r0, int i, int u, int c,
                                       const float (&v)[4]) {
  const int row = r0 + i;
  if (row >= g.rows) return;
  if (g.dest == kHeadFloatRows) {
    hp_store4(reinterpret_cast<float*>(g.out) + row * g.ld + u * g.dim + c, v);
  } else if (g.dest == kHeadRows) {
    hp_store4(reinterpret_cast<T*>(g.out) + row * g.ld + size_t(u) * g.HD + c, v);
  } else if (info.page[i] >= 0) {
    hp_store4(reinterpret_cast<T*>(g.out) + ((size_t(info.page[i]) * g.units + u) * p.block_size + info.off[i]) * g.HD + c, v);
  }
}

// The angles of N neighbouring pairs from j on, for the block's row i: from shared memory, or (TAB) from the step's table.
template <int N, bool TAB>
__device__ __forceinline__ void hp_angles(const HeadPrepareParams& p, const HeadSegment& g, const float* cs, int n_cs, int r0, int i, int j,
                                          float (&c)[N], float (&s)[N]) {
  const int t = g.table, half = p.half[t];
  if constexpr (TAB) {
    const float* at = p.cs[t] + size_t(min(r0 + i, p.rows - 1)) * 2 * half + j;
    if constexpr (N == 4) {
      hp_load4(c, at);
      hp_load4(s, at + half);
    } else {
#pragma unroll
      for (int e = 0; e < N; ++e) {
        const bool in = j + e < half;
        c[e] = in ? at[e] : 1.f;
        s[e] = in ? at[half + e] : 0.f;
      }
    }
#pragma unroll
    for (int e = 0; e < N; ++e) {
      c[e] *= p.amplitude[t];
      s[e] *= p.amplitude[t];
    }
  } else {
    const float* at = cs + i * n_cs + (t ? 2 * p.half[0] : 0) + j;
#pragma unroll
    for (int e = 0; e < N; ++e) {
      const bool in = j + e < half;
      c[e] = in ? at[e] : 1.f;
      s[e] = in ? at[half + e] : 0.f;
    }
  }
}

template <typename T, int TAPS, int R, bool TAB>
__global__ void __launch_bounds__(kHeadPrepareThreads, R > 1 ? 3 : 1)
head_prepare_kernel(const __grid_constant__ HeadPrepareParams p) {
  extern __shared__ __align__(16) float cs[];
  __shared__ HeadRowInfo<R> info;
  pdl_launch_dependents();
  const int r0 = blockIdx.x * R;
  if (threadIdx.x < R) {
    const int row = r0 + threadIdx.x;
    const bool in = row < p.rows;
    int local = 0, slot = -1;
    if (in && p.conv_w) {
      const int s = p.row_seq[row];
      local = row - p.seq_q_start[s];
      slot = p.seq_state_slot[s];
    }
    const int cache = in && p.slot_mapping ? p.slot_mapping[row] : -1;
    const int page = cache >= 0 ? cache / p.block_size : -1;
    info.local[threadIdx.x] = local;
    info.state_slot[threadIdx.x] = slot;
    info.page[threadIdx.x] = page;
    info.off[threadIdx.x] = cache - page * p.block_size;
    if constexpr (R > 1) {
      const unsigned mask = (1u << R) - 1;
      const bool all = __all_sync(mask, in && local >= TAPS - 1);
      if (threadIdx.x == 0) info.whole = all;
    }
  }
  if constexpr (!TAB) hp_tables<R>(p, r0, cs);
  __syncthreads();
  pdl_wait();
  const int n_cs = 2 * (p.half[0] + p.half[1]);
  for (int item = blockIdx.y * blockDim.x + threadIdx.x; item < p.items; item += gridDim.y * blockDim.x) {
    int s = 0, it = item;
    while (it >= p.seg[s].units * p.seg[s].items) { it -= p.seg[s].units * p.seg[s].items; ++s; }
    const HeadSegment& g = p.seg[s];
    if (r0 >= g.rows) continue;
    const int u = it / g.items, k = it - u * g.items;
    const int half = g.table >= 0 ? p.half[g.table] : 0;
    if (half > 0 && !g.interleaved && k < half / 4) {                   // four pairs (c, c + half)
      const int c = 4 * k;
      float a[R][4], b[R][4];
      hp_quads<TAPS, R>(p, g, info, r0, u, c, a);
      hp_quads<TAPS, R>(p, g, info, r0, u, c + half, b);
#pragma unroll
      for (int i = 0; i < R; ++i) {
        float x[4], y[4], co[4], si[4];
        hp_angles<4, TAB>(p, g, cs, n_cs, r0, i, c, co, si);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          rotate_pair(a[i][e], b[i][e], co[e], si[e], x[e], y[e]);
          x[e] *= g.scale;
          y[e] *= g.scale;
        }
        hp_put<T, R>(p, g, info, r0, i, u, c, x);
        hp_put<T, R>(p, g, info, r0, i, u, c + half, y);
      }
      continue;
    }
    const int c = half > 0 && !g.interleaved ? 2 * half + 4 * (k - half / 4) : 4 * k;
    float a[R][4];
    if (c < g.dim) {
      hp_quads<TAPS, R>(p, g, info, r0, u, c, a);
    } else {                                                             // the padding of a head
#pragma unroll
      for (int i = 0; i < R; ++i) a[i][0] = a[i][1] = a[i][2] = a[i][3] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
      if (half > 0 && g.interleaved && c < 2 * half) {
        float co[2], si[2];
        hp_angles<2, TAB>(p, g, cs, n_cs, r0, i, c / 2, co, si);
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          if (c / 2 + e / 2 >= half) break;
          float x, y;
          rotate_pair(a[i][e], a[i][e + 1], co[e / 2], si[e / 2], x, y);
          a[i][e] = x;
          a[i][e + 1] = y;
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) a[i][e] *= g.scale;
      hp_put<T, R>(p, g, info, r0, i, u, c, a[i]);
    }
  }
}

// One element of any size, one block a row; the state is left to the second launch.
__device__ __forceinline__ float hp_element(const HeadPrepareParams& p, const HeadSegment& g, int row, int local, int slot, int at) {
  const float* src = p.proj + row * p.ldp + g.src + at;
  if (g.conv < 0) return *src;
  float acc = 0.f;
  for (int j = 0; j < p.taps; ++j) {
    const int back = p.taps - 1 - j;
    float x = 0.f;
    if (local >= back) x = src[-back * p.ldp];
    else if (slot >= 0) x = p.state[slot * p.state_stride + (long long)(p.taps - 1 + local - back) * p.channels + g.conv + at];
    acc = fmaf(p.conv_w[size_t(g.conv + at) * p.taps + j], x, acc);
  }
  return acc;
}

// (Elements of one head are formed by one warp that holds all of them back until every lane has read its own: a segment
// may be written in place.)
template <typename T>
__global__ void __launch_bounds__(kHeadPrepareThreads)
head_prepare_any_kernel(const __grid_constant__ HeadPrepareParams p) {
  extern __shared__ __align__(16) float cs[];         // the row's cosines and sines, then a head's values for every warp
  pdl_launch_dependents();
  const int row = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  hp_tables<1>(p, row, cs);
  const int n_cs = 2 * (p.half[0] + p.half[1]);
  int widest = 0, heads = 0;
  for (int s = 0; s < p.segments; ++s) { widest = max(widest, p.seg[s].dim); heads += p.seg[s].units; }
  float* mine = cs + n_cs + warp * widest;
  int local = 0, slot = -1;
  if (p.conv_w) {
    const int q = p.row_seq[row];
    local = row - p.seq_q_start[q];
    slot = p.seq_state_slot[q];
  }
  const int cache = p.slot_mapping ? p.slot_mapping[row] : -1;
  __syncthreads();
  pdl_wait();
  for (int h = warp; h < heads; h += nwarps) {
    int s = 0, u = h;
    while (u >= p.seg[s].units) { u -= p.seg[s].units; ++s; }
    const HeadSegment& g = p.seg[s];
    if (row >= g.rows) continue;
    const int half = g.table >= 0 ? p.half[g.table] : 0;
    const float* table = cs + (g.table == 1 ? 2 * p.half[0] : 0);
    for (int c = lane; c < g.dim; c += 32) mine[c] = hp_element(p, g, row, local, slot, u * g.dim + c);
    __syncwarp();
    for (int j = lane; j < half; j += 32) {
      const int ia = g.interleaved ? 2 * j : j, ib = g.interleaved ? 2 * j + 1 : j + half;
      float x, y;
      rotate_pair(mine[ia], mine[ib], table[j], table[half + j], x, y);
      mine[ia] = x;
      mine[ib] = y;
    }
    __syncwarp();
    for (int c = lane; c < g.HD; c += 32) {
      const float v = c < g.dim ? mine[c] * g.scale : 0.f;
      if (g.dest == kHeadFloatRows) {
        reinterpret_cast<float*>(g.out)[row * g.ld + u * g.dim + c] = v;
      } else if (g.dest == kHeadRows) {
        stf(reinterpret_cast<T*>(g.out) + row * g.ld + size_t(u) * g.HD + c, v);
      } else if (cache >= 0) {
        const int page = cache / p.block_size, off = cache - page * p.block_size;
        stf(reinterpret_cast<T*>(g.out) + ((size_t(page) * g.units + u) * p.block_size + off) * g.HD + c, v);
      }
    }
    __syncwarp();
  }
}

// Behind the convolution: the state keeps the last taps - 1 inputs of every request.  One thread owns one (request, channel)
// and moves old entries down before it overwrites them.
__global__ void __launch_bounds__(256)
head_conv_state_kernel(const float* __restrict__ cols, long long ldp, int taps, float* __restrict__ state, long long state_stride,
                       const int* __restrict__ seq_q_start, const int* __restrict__ seq_q_len,
                       const int* __restrict__ seq_state_slot, int channels) {
  pdl_launch_dependents();
  const int s = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x, slot = seq_state_slot[s];
  const int q0 = seq_q_start[s], n = seq_q_len[s];
  pdl_wait();
  if (c >= channels || slot < 0) return;
  float* kept = state + slot * state_stride + c;
  for (int j = 0; j < taps - 1; ++j) {
    const int l = n - (taps - 1) + j;
    kept[(long long)j * channels] = l >= 0 ? cols[(q0 + l) * ldp + c] : kept[(long long)(n + j) * channels];
  }
}

template <typename T, int TAPS>
static int launch_head_prepare_quads(HeadPrepareParams p, cudaStream_t s) {
  const bool run = p.rows >= 1024;                             // many rows: several of them a thread
  const int R = run ? kHeadRunRows : 1;
  const int bx = (p.rows + R - 1) / R, most = (p.items + kHeadPrepareThreads - 1) / kHeadPrepareThreads;
  auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  bool tab = run;                                              // (every rotation of the launch has a table)
  for (int t = 0; t < 2; ++t) tab = tab && (p.half[t] == 0 || (p.cs[t] && (p.half[t] % 4) == 0 && aligned(p.cs[t])));
  const int by = tab ? most : max(1, min(most, 592 / bx));
  const size_t smem = tab ? 0 : size_t(R) * 2 * (p.half[0] + p.half[1]) * sizeof(float);
  if (tab) return pdl_launch(head_prepare_kernel<T, TAPS, kHeadRunRows, true>, dim3(bx, by), dim3(kHeadPrepareThreads), smem, s, p);
  if (run) return pdl_launch(head_prepare_kernel<T, TAPS, kHeadRunRows, false>, dim3(bx, by), dim3(kHeadPrepareThreads), smem, s, p);
  return pdl_launch(head_prepare_kernel<T, TAPS, 1, false>, dim3(bx, by), dim3(kHeadPrepareThreads), smem, s, p);
}

template <typename T>
static int launch_head_prepare(HeadPrepareParams p, cudaStream_t s) {
  if (p.rows == 0) return 0;
  if (p.segments < 1 || p.segments > kMaxHeadSegments || p.half[0] < 0 || p.half[1] < 0 || p.half[0] + p.half[1] > 4096 ||
      (p.conv_w && p.taps < 1))
    return KVCM_ERR_UNSUPPORTED;
  auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  bool quads = (p.ldp % 4) == 0 && aligned(p.proj) && (!p.conv_w || (p.taps <= 4 && (p.channels % 4) == 0 && (p.state_stride % 4) == 0 &&
                                                                     aligned(p.conv_w) && aligned(p.state)));
  int widest = 0;
  p.items = 0;
  for (int i = 0; i < p.segments; ++i) {
    HeadSegment& g = p.seg[i];
    if (g.units < 1 || g.dim < 1 || g.rows < 0 || g.rows > p.rows || g.HD < g.dim || g.table > 1 || (g.table >= 0 && 2 * p.half[g.table] > g.dim) ||
        (g.dest == kHeadFloatRows && g.HD != g.dim) || (g.conv >= 0 && !p.conv_w) || g.dest < 0 || g.dest > 2)
      return KVCM_ERR_UNSUPPORTED;
    const int half = g.table >= 0 ? p.half[g.table] : 0;
    quads = quads && (g.dim % 4) == 0 && (g.HD % 4) == 0 && (g.src % 4) == 0 && (g.conv < 0 || (g.conv % 4) == 0) && aligned(g.out) &&
            (g.dest == kHeadPages || (g.ld % 4) == 0) && (g.interleaved || (half % 4) == 0);
    g.items = half > 0 && !g.interleaved ? half / 4 + (g.HD - 2 * half) / 4 : g.HD / 4;
    p.items += g.units * g.items;
    widest = max(widest, g.dim);
  }
  const bool single = p.rows == p.seqs;
  p.write_state = quads && single && p.conv_w && p.taps > 1;
  int rc;
  if (quads) {
    switch (p.conv_w ? p.taps : 1) {
      case 1: rc = launch_head_prepare_quads<T, 1>(p, s); break;
      case 2: rc = launch_head_prepare_quads<T, 2>(p, s); break;
      case 3: rc = launch_head_prepare_quads<T, 3>(p, s); break;
      default: rc = launch_head_prepare_quads<T, 4>(p, s); break;
    }
  } else {
    const size_t smem = (2 * size_t(p.half[0] + p.half[1]) + size_t(kHeadPrepareThreads / 32) * widest) * sizeof(float);
    if (smem > 200 * 1024) return KVCM_ERR_UNSUPPORTED;
    if (smem > 48 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(head_prepare_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
      if (e != cudaSuccess) return int(e);
    }
    rc = pdl_launch(head_prepare_any_kernel<T>, dim3(p.rows), dim3(kHeadPrepareThreads), smem, s, p);
  }
  if (rc || !p.conv_w || p.taps < 2 || p.write_state) return rc;
  return pdl_launch(head_conv_state_kernel, dim3(p.seqs, (p.channels + 255) / 256), dim3(256), 0, s, p.proj + p.conv_col, p.ldp, p.taps,
                    p.state, p.state_stride, p.seq_q_start, p.seq_q_len, p.seq_state_slot, p.channels);
}

// ------------------------------------------------------------------------------------------ behind the mixers
//
// Heads on their way to an output product, for up to kMaxGateSegments runs of equal heads in one launch:
//   out = x [/ sqrt(mean_head(x^2) + eps)] * act(gate),   act = sigmoid | silu
// x is the attention kernel's output (storage type, padded heads) or a recurrence's (float); gate logits are float columns of
// the projection.  A warp takes a head.

constexpr int kMaxGateSegments = 4;
struct GateSegment {                       // (mirrored by kernels/library.py)
  const void* x; void* out; long long ldx, ldo;
  int x_float, heads, dv, HD;              // HD: elements from one head of x to the next
  int gate, norm, silu;                    // first gate column
  float eps;
};
struct HeadGateParams {
  const float* gates; long long ldg;
  int rows, segments, heads, vec;
  GateSegment seg[kMaxGateSegments];
};

template <typename T>
__device__ __forceinline__ float hg_at(const GateSegment& g, size_t at) {
  return g.x_float ? reinterpret_cast<const float*>(g.x)[at] : ldf(reinterpret_cast<const T*>(g.x) + at);
}
template <typename T>
__device__ __forceinline__ void hg_load4(const GateSegment& g, size_t at, float (&v)[4]) {
  if (sizeof(T) == 4 || g.x_float) {
    hp_load4(v, reinterpret_cast<const float*>(g.x) + at);
  } else {
    const uint2 raw = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(g.x) + at);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
head_gate_kernel(const __grid_constant__ HeadGateParams p) {
  pdl_launch_dependents();
  const int row = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  pdl_wait();
  for (int h = blockIdx.y * nwarps + warp; h < p.heads; h += gridDim.y * nwarps) {
    int s = 0, u = h;
    while (u >= p.seg[s].heads) { u -= p.seg[s].heads; ++s; }
    const GateSegment& g = p.seg[s];
    const size_t at = size_t(row) * g.ldx + size_t(u) * g.HD;
    const float* gate = p.gates + row * p.ldg + g.gate + u * g.dv;
    T* out = reinterpret_cast<T*>(g.out) + size_t(row) * g.ldo + size_t(u) * g.dv;
    // (bfloat16 results: CUDA's fast exponential and division, a few units in float's last place)
    auto act = [&](float z) {
      const float sg = sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-z)) : 1.f / (1.f + expf(-z));
      return g.silu ? z * sg : sg;
    };
    if (p.vec && g.dv <= 256) {                       // up to two quads a lane, kept in registers between the two passes
      float x[2][4], z[2][4];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int c = 4 * lane + 128 * k;
        x[k][0] = x[k][1] = x[k][2] = x[k][3] = 0.f;
        if (c < g.dv) { hg_load4<T>(g, at + c, x[k]); hp_load4(z[k], gate + c); }
      }
      float inv = 1.f;
      if (g.norm) {
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < 2; ++k)
#pragma unroll
          for (int e = 0; e < 4; ++e) ss = fmaf(x[k][e], x[k][e], ss);
        inv = 1.f / sqrtf(warp_sum(ss) / float(g.dv) + g.eps);
      }
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int c = 4 * lane + 128 * k;
        if (c >= g.dv) break;
        float y[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] = x[k][e] * inv * act(z[k][e]);
        hp_store4(out + c, y);
      }
      continue;
    }
    float inv = 1.f;
    if (g.norm) {
      float ss = 0.f;
      for (int c = lane; c < g.dv; c += 32) { const float v = hg_at<T>(g, at + c); ss = fmaf(v, v, ss); }
      inv = 1.f / sqrtf(warp_sum(ss) / float(g.dv) + g.eps);
    }
    for (int c = lane; c < g.dv; c += 32) stf(out + c, hg_at<T>(g, at + c) * inv * act(gate[c]));
  }
}

template <typename T>
static int launch_head_gate(HeadGateParams p, cudaStream_t s) {
  if (p.rows == 0) return 0;
  if (p.segments < 1 || p.segments > kMaxGateSegments) return KVCM_ERR_UNSUPPORTED;
  auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  p.vec = (p.ldg % 4) == 0 && aligned(p.gates);
  p.heads = 0;
  for (int i = 0; i < p.segments; ++i) {
    const GateSegment& g = p.seg[i];
    if (g.heads < 1 || g.dv < 1 || g.HD < g.dv) return KVCM_ERR_UNSUPPORTED;
    p.vec = p.vec && aligned(g.x) && aligned(g.out) && (g.dv % 4) == 0 && (g.HD % 4) == 0 && (g.ldx % 4) == 0 && (g.ldo % 4) == 0 && (g.gate % 4) == 0;
    p.heads += g.heads;
  }
  const int by = max(1, min((p.heads + 7) / 8, 1184 / p.rows));
  return pdl_launch(head_gate_kernel<T>, dim3(p.rows, by), dim3(256), 0, s, p);
}

}  // namespace kvcm

using namespace kvcm;

// The parameter blocks are passed by address (they are copied into the launch); `items`, `heads`, `vec` and `write_state` are filled in here.
KVCM_API int kvcm_head_prepare_params_bytes(void) { return int(sizeof(HeadPrepareParams)); }
KVCM_API int kvcm_head_prepare_f32(const void* params, void* stream) {
  return launch_head_prepare<float>(*static_cast<const HeadPrepareParams*>(params), (cudaStream_t)stream);
}
KVCM_API int kvcm_head_prepare_bf16(const void* params, void* stream) {
  return launch_head_prepare<bf16>(*static_cast<const HeadPrepareParams*>(params), (cudaStream_t)stream);
}
KVCM_API int kvcm_head_gate_params_bytes(void) { return int(sizeof(HeadGateParams)); }
KVCM_API int kvcm_head_gate_f32(const void* params, void* stream) {
  return launch_head_gate<float>(*static_cast<const HeadGateParams*>(params), (cudaStream_t)stream);
}
KVCM_API int kvcm_head_gate_bf16(const void* params, void* stream) {
  return launch_head_gate<bf16>(*static_cast<const HeadGateParams*>(params), (cudaStream_t)stream);
}
