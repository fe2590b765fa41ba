// Time mixing: a linear recurrence whose decays are made from the token, with a bonus for the current token, in 32-bit
// arithmetic whatever the storage type, and the blends of a token's row with the row before it that it reads.
//
//   token_shift: out_s[r] = h[r] + (h[r - 1] - h[r]) * mu_s for every blend s, side by side; the row before a segment's
//   first row is the last row of the request's step before (part of its state; zeros at the start of a sequence).
//
//   time_mixing: per request and head the state is a matrix S [D key channels x D value columns], zero at the start.
//   For every token, in order, with w = exp(-exp(raw + w0)) per key channel:
//     o = (S + diag(u) k v^T)^T r;   S <- diag(w) S + k v^T
//   The decay is used as 1 - w = -expm1(-exp(raw + w0)): S - (1 - w) S keeps the digits of a decay near 1 that the
//   rounded decay itself has lost.  The bonus is one number per token and head, (sum over d of r_d u_d k_d) v.
//   A segment's rows are walked in order from the request's state, so a position's values do not depend on how its
//   prompt was cut beyond rounding.
//
// grid (column blocks, heads, segments).  A block owns CB columns of S; a thread holds CPT of them (4, 2 where a column is
// long, 1 in steps of short segments), each spread over L lanes: a lane holds runs of four channels, 4 l + 4 L i on, in
// registers, so its share of a row staged in shared memory is read 16 bytes at a time without bank conflicts and serves CPT
// columns.  Rows come through shared memory TC at a time (keys, receptances, 1 - w, the block's slice of values); the next
// TC rows are on their way from memory, into registers, while these are walked.  (Packed 32-bit multiply-adds and
// fetching entries in pairs were tried: no faster where the walk is cut into pieces, 1.4 times slower where it is not.)
//
// One long prompt offers heads x columns of parallel work only.  Where a step's states are few and its longest segment is
// long, segments are cut into pieces of `piece_rows` rows that run side by side, in three launches: every piece but a
// segment's last walks its rows from a zero state and leaves the end state and the product of its decays per channel; the
// start states follow one after the other, start[p + 1] = product_p start[p] + end_p, start[0] the request's state; then
// every piece walks its rows again from its start state and writes its results, the last piece the request's state.
#include "common.cuh"

namespace cbis {

constexpr int kMixRows = 16;       // rows of a batch for long segments
constexpr int kMixRowsShort = 4;   // rows of a batch where no segment of the step is longer (decode steps)
constexpr int kShiftMost = 8;      // blends token_shift takes

enum { kMixWhole = 0, kMixEnds = 1, kMixFromStarts = 2 };

template <typename TT, int V>
struct alignas(sizeof(TT) * V) Run {
  TT e[V];
};

// grid (runs of `run` rows, blocks of columns); a thread takes V columns of every row of the run, with the blends' weights of
// these columns in registers, and asks for the next row while it works on one.  The thread that meets a segment's first row
// reads the row kept in the state and then replaces it by the segment's last row: no other thread touches these columns of it.
template <typename TT, int V, int N>
__global__ void __launch_bounds__(256)
token_shift_kernel(const TT* h, int ld, float* state, long long slot_stride, const int* seg_slot, const int* row_seq,
                   const int* cu_rows, const float* __restrict__ mu, int n_mix, TT* out, int out_ld, int width, int rows, int run) {
  pdl_trigger();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= width) return;
  float m[N][V];
#pragma unroll
  for (int s = 0; s < N; ++s)
#pragma unroll
    for (int k = 0; k < V; ++k) m[s][k] = s < n_mix ? mu[(size_t)s * width + c + k] : 0.f;
  pdl_wait();
  const int r0 = blockIdx.x * run, r1 = min(rows, r0 + run);
  float prev[V];
  int have = -1;                       // the row whose values prev holds
  Run<TT, V> next = *reinterpret_cast<const Run<TT, V>*>(h + (size_t)r0 * ld + c);
  for (int r = r0; r < r1; ++r) {
    const int seq = row_seq[r];
    const Run<TT, V> now = next;
    if (r + 1 < r1) next = *reinterpret_cast<const Run<TT, V>*>(h + (size_t)(r + 1) * ld + c);
    TT* o = out + (size_t)r * out_ld + c;
    if (seq < 0) {                     // a padding row of a fixed-size batch
      Run<TT, V> z;
#pragma unroll
      for (int k = 0; k < V; ++k) from_f32(z.e[k], 0.f);
      for (int s = 0; s < n_mix; ++s) *reinterpret_cast<Run<TT, V>*>(o + (size_t)s * width) = z;
      continue;
    }
    float x[V];
#pragma unroll
    for (int k = 0; k < V; ++k) x[k] = to_f32(now.e[k]);
    if (r == cu_rows[seq]) {
      float* kept = state + (long long)seg_slot[seq] * slot_stride + c;
      const Run<TT, V> last = *reinterpret_cast<const Run<TT, V>*>(h + (size_t)(cu_rows[seq + 1] - 1) * ld + c);
#pragma unroll
      for (int k = 0; k < V; ++k) {
        prev[k] = kept[k];
        kept[k] = to_f32(last.e[k]);
      }
    } else if (have != r - 1) {
      const Run<TT, V> b = *reinterpret_cast<const Run<TT, V>*>(h + (size_t)(r - 1) * ld + c);
#pragma unroll
      for (int k = 0; k < V; ++k) prev[k] = to_f32(b.e[k]);
    }
#pragma unroll
    for (int s = 0; s < N; ++s) {
      if (s < n_mix) {
        Run<TT, V> b;
#pragma unroll
        for (int k = 0; k < V; ++k) from_f32(b.e[k], fmaf(prev[k] - x[k], m[s][k], x[k]));
        *reinterpret_cast<Run<TT, V>*>(o + (size_t)s * width) = b;
      }
    }
#pragma unroll
    for (int k = 0; k < V; ++k) prev[k] = x[k];
    have = r;
  }
}

template <typename TT, int NPL, int L, int CPT, int CB, int TC, int MODE>
__global__ void __launch_bounds__(CB / CPT * L)
time_mixing_kernel(const TT* x, int ld, int r_off, int k_off, int v_off, const float* raw, int raw_ld,
                   const float* __restrict__ w0, const float* __restrict__ u, float* state, long long slot_stride,
                   const int* seg_slot, const int* cu_rows, float* y, int y_ld, int H, int D, int n_pieces, int piece_rows,
                   float* starts, float* products) {
  static_assert(NPL % 4 == 0 && (CPT == 1 || CPT == 2 || CPT == 4), "channels a lane in runs of four; columns a thread");
  constexpr int DP = NPL * L, THREADS = CB / CPT * L, RUNS = NPL / 4;
  constexpr int PER = (TC * DP + THREADS - 1) / THREADS, V_PER = (TC * CB + THREADS - 1) / THREADS;
  extern __shared__ __align__(16) float smem[];
  float* ks = smem;                  // [TC][DP]
  float* os = ks + TC * DP;          // [TC][DP]: 1 - w
  float* rs = os + TC * DP;          // [TC][DP]
  float* vs = rs + TC * DP;          // [TC][CB]
  float* nums = vs + TC * CB;        // [TC][CB]
  float* bonus = nums + TC * CB;     // [TC]
  pdl_trigger();
  const int xb = blockIdx.x, h = blockIdx.y;
  int s = blockIdx.z, piece = 0;
  if (MODE != kMixWhole) {
    piece = s % n_pieces;
    s /= n_pieces;
  }
  pdl_wait();
  int row0 = cu_rows[s], n_rows = cu_rows[s + 1] - row0;
  bool last = true;                  // the piece that holds the segment's last row leaves the request's state
  if (MODE != kMixWhole) {
    const int before = piece * piece_rows;
    last = before + piece_rows >= n_rows;
    if (before >= n_rows || (MODE == kMixEnds && last)) return;
    row0 += before;
    n_rows = min(piece_rows, n_rows - before);
  }
  if (n_rows <= 0) return;
  const int tid = threadIdx.x;
  const int l = tid % L, g = tid / L;
  const int col = xb * CB + g * CPT;           // the first of this thread's columns
  const size_t at = ((size_t)h * D + (col < D ? col : 0)) * D;       // its place in a state
  const size_t per_state = (size_t)H * D * D;
  float* sp = state + (long long)seg_slot[s] * slot_stride + at;
  const float* from = MODE == kMixFromStarts ? starts + ((size_t)s * n_pieces + piece) * per_state + at : sp;
  float* into = MODE == kMixEnds ? starts + ((size_t)s * n_pieces + piece + 1) * per_state + at : sp;
  auto channel = [&](int i) { return (i >> 2) * 4 * L + 4 * l + (i & 3); };      // of this lane's entry i
  const bool by4 = D % 4 == 0 && slot_stride % 4 == 0;      // a lane's runs lie whole in a column, 16-byte aligned
  float S[CPT][NPL], P[MODE == kMixEnds ? NPL : 1];
#pragma unroll
  for (int j = 0; j < CPT; ++j) {
#pragma unroll
    for (int q = 0; q < RUNS; ++q) {
      const int d = channel(4 * q);
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      if (MODE != kMixEnds && col + j < D) {
        const float* p = from + (size_t)j * D + d;
        if (by4) {
          if (d < D) a = *reinterpret_cast<const float4*>(p);
        } else {
          if (d < D) a.x = p[0];
          if (d + 1 < D) a.y = p[1];
          if (d + 2 < D) a.z = p[2];
          if (d + 3 < D) a.w = p[3];
        }
      }
      S[j][4 * q] = a.x, S[j][4 * q + 1] = a.y, S[j][4 * q + 2] = a.z, S[j][4 * q + 3] = a.w;
    }
  }
  if constexpr (MODE == kMixEnds) {
#pragma unroll
    for (int i = 0; i < NPL; ++i) P[i] = 1.f;
  }
  const TT* rrow = x + (size_t)row0 * ld + r_off + h * D;
  const TT* krow = x + (size_t)row0 * ld + k_off + h * D;
  const TT* vrow = x + (size_t)row0 * ld + v_off + h * D + xb * CB;
  const float* wrow = raw + (size_t)row0 * raw_ld + h * D;
  const int vcols = min(CB, D - xb * CB);

  // what this thread fetches of a batch of rows: entries of k, r and the raw decays (row t = idx / DP, channel d =
  // idx % DP) and of the block's slice of v
  float f_k[PER], f_r[PER], f_w[PER], f_v[V_PER];
  auto fetch = [&](int first) {
    const int tc = min(TC, n_rows - first);
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int idx = tid + THREADS * j, t = idx / DP, d = idx % DP;
      const bool ok = t < tc && d < D;
      f_k[j] = ok ? to_f32(krow[(size_t)(first + t) * ld + d]) : 0.f;
      f_w[j] = ok ? wrow[(size_t)(first + t) * raw_ld + d] : 0.f;
      f_r[j] = (MODE != kMixEnds && ok) ? to_f32(rrow[(size_t)(first + t) * ld + d]) : 0.f;
    }
#pragma unroll
    for (int j = 0; j < V_PER; ++j) {
      const int idx = tid + THREADS * j, t = idx / CB, cc = idx % CB;
      f_v[j] = (t < tc && cc < vcols) ? to_f32(vrow[(size_t)(first + t) * ld + cc]) : 0.f;
    }
  };
  fetch(0);
  for (int first = 0; first < n_rows; first += TC) {
    const int tc = min(TC, n_rows - first);
    __syncthreads();                 // the rows staged before have been used
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int idx = tid + THREADS * j, d = idx % DP;
      if (idx < TC * DP) {
        ks[idx] = f_k[j];
        os[idx] = d < D ? -expm1f(-expf(f_w[j] + w0[h * D + d])) : 0.f;
        if (MODE != kMixEnds) rs[idx] = f_r[j];
      }
    }
#pragma unroll
    for (int j = 0; j < V_PER; ++j) {
      const int idx = tid + THREADS * j;
      if (idx < TC * CB) vs[idx] = f_v[j];
    }
    __syncthreads();
    if (first + TC < n_rows) fetch(first + TC);      // in flight while these rows are walked
    if (MODE != kMixEnds) {          // a warp per row: the bonus
      for (int t = tid >> 5; t < tc; t += THREADS / 32) {
        float b = 0.f;
        for (int d = tid & 31; d < D; d += 32) b = fmaf(rs[t * DP + d] * u[h * D + d], ks[t * DP + d], b);
        b = warp_sum(b);
        if ((tid & 31) == 0) bonus[t] = b;
      }
    }
#pragma unroll 2
    for (int t = 0; t < tc; ++t) {
      float kk[NPL], oo[NPL], rr[NPL], vv[CPT];
#pragma unroll
      for (int q = 0; q < RUNS; ++q) {
        const int d = t * DP + channel(4 * q);
        const float4 a = *reinterpret_cast<const float4*>(ks + d), b = *reinterpret_cast<const float4*>(os + d);
        kk[4 * q] = a.x, kk[4 * q + 1] = a.y, kk[4 * q + 2] = a.z, kk[4 * q + 3] = a.w;
        oo[4 * q] = b.x, oo[4 * q + 1] = b.y, oo[4 * q + 2] = b.z, oo[4 * q + 3] = b.w;
        if (MODE != kMixEnds) {
          const float4 c = *reinterpret_cast<const float4*>(rs + d);
          rr[4 * q] = c.x, rr[4 * q + 1] = c.y, rr[4 * q + 2] = c.z, rr[4 * q + 3] = c.w;
        }
      }
      if constexpr (CPT == 4) {
        const float4 a = *reinterpret_cast<const float4*>(vs + t * CB + g * 4);
        vv[0] = a.x, vv[1] = a.y, vv[2] = a.z, vv[3] = a.w;
      } else if constexpr (CPT == 2) {
        const float2 a = *reinterpret_cast<const float2*>(vs + t * CB + g * 2);
        vv[0] = a.x, vv[1] = a.y;
      } else {
        vv[0] = vs[t * CB + g];
      }
      if constexpr (MODE == kMixEnds) {          // the end state and the decays' product only
#pragma unroll
        for (int i = 0; i < NPL; ++i) {
          P[i] = fmaf(-oo[i], P[i], P[i]);
#pragma unroll
          for (int j = 0; j < CPT; ++j) S[j][i] = fmaf(vv[j], kk[i], fmaf(-oo[i], S[j][i], S[j][i]));
        }
      } else {
        float a0[CPT], a1[CPT], acc[CPT];
#pragma unroll
        for (int j = 0; j < CPT; ++j) a0[j] = a1[j] = 0.f;
#pragma unroll
        for (int i = 0; i < NPL; ++i) {
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            if (i & 1) a1[j] = fmaf(S[j][i], rr[i], a1[j]);
            else a0[j] = fmaf(S[j][i], rr[i], a0[j]);
            S[j][i] = fmaf(vv[j], kk[i], fmaf(-oo[i], S[j][i], S[j][i]));
          }
        }
#pragma unroll
        for (int j = 0; j < CPT; ++j) acc[j] = a0[j] + a1[j];
        // the sum over a column's lanes; a lane passes on the columns its partner keeps
        float sum;
        int mine = 0, o = 1;                       // the column (of CPT) whose sum this lane ends with
        if constexpr (CPT == 4) {
          const bool hi = l & 1, hi2 = l & 2;
          float k0 = hi ? acc[2] : acc[0], k1 = hi ? acc[3] : acc[1];
          k0 += __shfl_xor_sync(0xffffffffu, hi ? acc[0] : acc[2], 1);
          k1 += __shfl_xor_sync(0xffffffffu, hi ? acc[1] : acc[3], 1);
          sum = (hi2 ? k1 : k0) + __shfl_xor_sync(0xffffffffu, hi2 ? k0 : k1, 2);
          mine = 2 * (l & 1) + ((l >> 1) & 1);
          o = 4;
        } else if constexpr (CPT == 2) {
          const bool hi = l & 1;
          sum = (hi ? acc[1] : acc[0]) + __shfl_xor_sync(0xffffffffu, hi ? acc[0] : acc[1], 1);
          mine = l & 1;
          o = 2;
        } else {
          sum = acc[0];
        }
#pragma unroll
        for (; o < L; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        if (l < CPT) nums[t * CB + g * CPT + mine] = sum;
      }
    }
    if constexpr (MODE != kMixEnds) {
      __syncthreads();
      for (int i = tid; i < tc * CB; i += THREADS) {
        const int t = i / CB, cc = i % CB;
        if (cc < vcols) y[(size_t)(row0 + first + t) * y_ld + h * D + xb * CB + cc] = fmaf(bonus[t], vs[i], nums[i]);
      }
    }
  }
  if (MODE != kMixFromStarts || last) {
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
#pragma unroll
      for (int q = 0; q < RUNS; ++q) {
        const int d = channel(4 * q);
        if (col + j < D) {
          float* p = into + (size_t)j * D + d;
          if (by4) {
            if (d < D) *reinterpret_cast<float4*>(p) = make_float4(S[j][4 * q], S[j][4 * q + 1], S[j][4 * q + 2], S[j][4 * q + 3]);
          } else {
#pragma unroll
            for (int k = 0; k < 4; ++k)
              if (d + k < D) p[k] = S[j][4 * q + k];
          }
        }
      }
    }
  }
  if constexpr (MODE == kMixEnds) {
    if (xb == 0 && g == 0) {         // the first column's lanes leave the products of the piece's decays
      float* pr = products + (((size_t)s * n_pieces + piece) * H + h) * D;
#pragma unroll
      for (int i = 0; i < NPL; ++i)
        if (channel(i) < D) pr[channel(i)] = P[i];
    }
  }
}

// The start states of a cut segment's pieces, one after the other: starts[s][0] is the request's state, starts[s][p]
// (which holds the end state, from zero, of piece p - 1) becomes products[s][p - 1] * starts[s][p - 1] + itself.
// grid (blocks of elements, segments); a thread owns one element of the state.
__global__ void __launch_bounds__(256)
time_mixing_starts_kernel(float* starts, const float* products, const float* state, long long slot_stride, const int* seg_slot,
                          const int* cu_rows, int n_pieces, int piece_rows, int H, int D) {
  pdl_trigger();
  pdl_wait();
  const int HDD = H * D * D, HD = H * D;
  const int s = blockIdx.y, e = blockIdx.x * blockDim.x + threadIdx.x;
  const int n_rows = cu_rows[s + 1] - cu_rows[s];
  if (e >= HDD || n_rows <= 0) return;
  const int np = (n_rows + piece_rows - 1) / piece_rows;
  const int c = e / (D * D) * D + e % D;                 // the element's channel among all heads'
  float* st = starts + (size_t)s * n_pieces * HDD + e;
  const float* pr = products + (size_t)s * n_pieces * HD + c;
  float cur = state[(long long)seg_slot[s] * slot_stride + e];
  st[0] = cur;
  int p = 1;
  for (; p + 4 <= np; p += 4) {       // four ends and products on their way at a time
    float en[4], de[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      en[k] = st[(size_t)(p + k) * HDD];
      de[k] = pr[(size_t)(p + k - 1) * HD];
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) st[(size_t)(p + k) * HDD] = cur = fmaf(de[k], cur, en[k]);
  }
  for (; p < np; ++p) st[(size_t)p * HDD] = cur = fmaf(pr[(size_t)(p - 1) * HD], cur, st[(size_t)p * HDD]);
}

template <typename TT>
static int launch_time_mixing(const void* x, int ld, int r_off, int k_off, int v_off, const float* raw, int raw_ld,
                              const float* w0, const float* u, float* state, long long slot_stride, const int* seg_slot,
                              const int* cu_rows, float* y, int y_ld, int S, int H, int D, int max_seg_rows, int n_pieces,
                              int piece_rows, float* starts, float* products, cudaStream_t st) {
  const bool shorts = max_seg_rows > 0 && max_seg_rows <= kMixRowsShort;
#define CBIS_MIX_AS(NPL, LL, CPT, TCC, MODE, Z)                                                                       \
  do {                                                                                                                \
    constexpr int CBB = CPT == 1 ? 32 : 16 * CPT;                                                                     \
    const size_t smem = ((size_t)3 * TCC * NPL * LL + 2 * TCC * CBB + TCC) * sizeof(float);                           \
    if (smem > 48 * 1024)                                                                                             \
      cudaFuncSetAttribute(time_mixing_kernel<TT, NPL, LL, CPT, CBB, TCC, MODE>,                                      \
                           cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                                   \
    err = launch_pdl(time_mixing_kernel<TT, NPL, LL, CPT, CBB, TCC, MODE>, dim3((D + CBB - 1) / CBB, H, Z),           \
                     dim3(CBB / CPT * LL), smem, st, (const TT*)x, ld, r_off, k_off, v_off, raw, raw_ld, w0, u, state, \
                     slot_stride, seg_slot, cu_rows, y, y_ld, H, D, n_pieces, piece_rows, starts, products);          \
  } while (0)
#define CBIS_MIX(NPL, LL)                                                                                             \
  do {                                                                                                                \
    cudaError_t err = cudaSuccess;                                                                                    \
    constexpr int CPT = NPL <= 16 ? 4 : 2;                                                                            \
    if (n_pieces > 1) {                                                                                               \
      CBIS_MIX_AS(NPL, LL, CPT, kMixRows, kMixEnds, S * n_pieces);                                                    \
      if (err != cudaSuccess) return (int)err;                                                                        \
      err = launch_pdl(time_mixing_starts_kernel, dim3((H * D * D + 255) / 256, S), dim3(256), 0, st, starts,         \
                       (const float*)products, (const float*)state, slot_stride, seg_slot, cu_rows, n_pieces,         \
                       piece_rows, H, D);                                                                             \
      if (err != cudaSuccess) return (int)err;                                                                        \
      CBIS_MIX_AS(NPL, LL, CPT, kMixRows, kMixFromStarts, S * n_pieces);                                              \
      return (int)err;                                                                                                \
    }                                                                                                                 \
    if (shorts) {                                                                                                     \
      CBIS_MIX_AS(NPL, LL, 1, kMixRowsShort, kMixWhole, S);                                                           \
      return (int)err;                                                                                                \
    }                                                                                                                 \
    CBIS_MIX_AS(NPL, LL, CPT, kMixRows, kMixWhole, S);                                                                \
    return (int)err;                                                                                                  \
  } while (0)
  if (D <= 32) CBIS_MIX(4, 8);
  if (D <= 64) CBIS_MIX(8, 8);
  if (D <= 96) CBIS_MIX(12, 8);
  if (D <= 128) CBIS_MIX(16, 8);
  if (D <= 256) CBIS_MIX(32, 8);
  CBIS_MIX(32, 16);
#undef CBIS_MIX
#undef CBIS_MIX_AS
}

template <typename TT, int V>
static int launch_token_shift(const void* h, int ld, float* state, long long slot_stride, const int* seg_slot,
                              const int* row_seq, const int* cu_rows, const float* mu, int n_mix, void* out, int out_ld,
                              int width, int rows, cudaStream_t st) {
  // few rows: a row a block, narrow blocks; many: runs of rows, so that the blends' weights are read once per run
  const int cols = (width + V - 1) / V, run = rows <= 256 ? 1 : 4;
  const int threads = rows <= 256 ? 64 : (cols >= 256 ? 256 : (cols >= 128 ? 128 : 64));
  const dim3 grid((rows + run - 1) / run, (cols + threads - 1) / threads);
  auto kern = n_mix <= 5 ? token_shift_kernel<TT, V, 5> : token_shift_kernel<TT, V, kShiftMost>;
  return (int)launch_pdl(kern, grid, dim3(threads), 0, st, (const TT*)h, ld, state, slot_stride, seg_slot, row_seq, cu_rows,
                         mu, n_mix, (TT*)out, out_ld, width, rows, run);
}

}  // namespace cbis

using namespace cbis;

CBIS_EXPORT int cbis_time_mixing_max_dim() { return 512; }

// h [rows, ld] and out [rows, out_ld] (n_mix * width columns) of the compute type; mu [n_mix, width] 32-bit; the row before
// a segment's first one: width 32-bit numbers at `state + slot * slot_stride`, replaced by the segment's last row.
CBIS_EXPORT int cbis_token_shift(const void* h, int ld, float* state, long long slot_stride, const int* seg_slot,
                                 const int* row_seq, const int* cu_rows, const float* mu, int n_mix, void* out, int out_ld,
                                 int width, int rows, int dtype, void* stream) {
  if (rows <= 0 || width <= 0) return CBIS_OK;
  if (n_mix <= 0 || n_mix > kShiftMost || out_ld < n_mix * width) return CBIS_ERR_BAD_SIZE;
  cudaStream_t st = (cudaStream_t)stream;
  const int v = dtype == CBIS_BF16 ? 8 : 4;
  const bool wide = width % v == 0 && ld % v == 0 && out_ld % v == 0 && !(((uintptr_t)h | (uintptr_t)out) & 15);
  if (dtype == CBIS_F32)
    return wide ? launch_token_shift<float, 4>(h, ld, state, slot_stride, seg_slot, row_seq, cu_rows, mu, n_mix, out, out_ld, width, rows, st)
                : launch_token_shift<float, 1>(h, ld, state, slot_stride, seg_slot, row_seq, cu_rows, mu, n_mix, out, out_ld, width, rows, st);
  if (dtype == CBIS_BF16)
    return wide ? launch_token_shift<__nv_bfloat16, 8>(h, ld, state, slot_stride, seg_slot, row_seq, cu_rows, mu, n_mix, out, out_ld, width, rows, st)
                : launch_token_shift<__nv_bfloat16, 1>(h, ld, state, slot_stride, seg_slot, row_seq, cu_rows, mu, n_mix, out, out_ld, width, rows, st);
  return CBIS_ERR_BAD_DTYPE;
}

// x [T, ld] of the compute type: r at columns r_off + h * D, k at k_off + h * D, v at v_off + h * D; raw [T, raw_ld] 32-bit,
// H * D columns; w0, u [H * D] 32-bit; max_seg_rows: the longest segment of the step (0: unknown); y [T, y_ld] 32-bit, H * D
// columns; state: 32-bit, H * D * D per slot ([head][value column][key channel]) at `state + slot * slot_stride`.
// n_pieces > 1: segments are cut into up to n_pieces pieces of piece_rows rows (a multiple of 16, and n_pieces * piece_rows
// >= max_seg_rows); starts: 32-bit scratch [n_segments * n_pieces][H * D * D], products: [n_segments * n_pieces][H * D].
CBIS_EXPORT int cbis_time_mixing(const void* x, int ld, int r_off, int k_off, int v_off, const float* raw, int raw_ld,
                                 const float* w0, const float* u, float* state, long long slot_stride, const int* seg_slot,
                                 const int* cu_rows, float* y, int y_ld, int n_segments, int H, int D, int dtype,
                                 void* stream, int max_seg_rows, int n_pieces, int piece_rows, float* starts,
                                 float* products) {
  if (n_segments <= 0) return CBIS_OK;
  if (H <= 0 || D <= 0 || D > 512) return CBIS_ERR_BAD_SIZE;
  if (n_segments > 65535 || H > 65535) return CBIS_ERR_TOO_LARGE;
  if (((uintptr_t)state & 15) || ((uintptr_t)starts & 15)) return CBIS_ERR_ALIGNMENT;
  if (n_pieces > 1) {
    if (piece_rows <= 0 || piece_rows % kMixRows || !starts || !products || max_seg_rows <= 0 ||
        (long long)n_pieces * piece_rows < max_seg_rows)
      return CBIS_ERR_BAD_SIZE;
    if ((long long)n_segments * n_pieces > 65535) return CBIS_ERR_TOO_LARGE;
  } else {
    n_pieces = 1;
  }
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == CBIS_F32)
    return launch_time_mixing<float>(x, ld, r_off, k_off, v_off, raw, raw_ld, w0, u, state, slot_stride, seg_slot, cu_rows, y,
                                     y_ld, n_segments, H, D, max_seg_rows, n_pieces, piece_rows, starts, products, st);
  if (dtype == CBIS_BF16)
    return launch_time_mixing<__nv_bfloat16>(x, ld, r_off, k_off, v_off, raw, raw_ld, w0, u, state, slot_stride, seg_slot,
                                             cu_rows, y, y_ld, n_segments, H, D, max_seg_rows, n_pieces, piece_rows, starts,
                                             products, st);
  return CBIS_ERR_BAD_DTYPE;
}
