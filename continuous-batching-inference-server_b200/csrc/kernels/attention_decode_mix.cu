// Decode attention (one query token a row, bfloat16) whose softmax weights are mixed across heads before they meet the
// values: w'_h(j) = sum_g T[h, g] w_g(j), out_h = sum_j w'_h(j) v_{kv(h)}(j), with an optional sink per head in the
// denominators and an optional gate on the result, element by element.
//
// A head's mixed weights need every head's finished denominator, so the keys are walked by two kernels:
//   * mix_scores: (row, key head, split of the keys): the scores of the query heads that share the key head, on the
//     tensor cores (mma.sync m16n8k16: the heads are the rows of A, 16 keys of B; both operands' K order permuted alike, so
//     that a 16-byte load of a key is two B fragments), scaled, into scratch memory in 32-bit, with the running maximum and
//     sum of every head; it also stores the current token's key;
//   * mix_values: (row, value head, split): all heads' weights of 128 keys at a time from the scores, mixed in 32-bit by one
//     thread a key, then the values times the mixed weights of the heads that read them; splits are plain sums (the
//     weights are finished), the block that comes last adds them up, applies the gate and rounds once; it also stores the
//     current token's value.
// Keys and values are each read once per row; what goes through scratch is H numbers a key.
#include "attention_decode_tc.cuh"
#include <math.h>

namespace cbis {

constexpr int MIX_KEYS = 128;      // keys a block of mix_values takes at a time

struct MixSplit {
  int kstart, kend, per;
};
// Keys of a row for `nsplit` splits: whole groups of 32 counted from the 16-key tile that holds the first key seen.
__device__ __forceinline__ MixSplit mix_split(int pos, int window, int nsplit) {
  MixSplit s;
  s.kend = pos + 1;
  s.kstart = first_seen(pos, window);
  const int from = s.kstart & ~15;
  s.per = (((s.kend - from) + nsplit - 1) / nsplit + 31) & ~31;
  return s;
}

// grid (rows, n_kv_head, nsplit).  NC: 32-entry pieces of a head (the last may be partly beyond it: read as zeros).
template <int NC>
__global__ void __launch_bounds__(DEC_WARPS * 32)
mix_scores_kernel(const __nv_bfloat16* qkv, int ld, int k_off, __nv_bfloat16* kc, const int* block_table, int max_blocks,
                  const int* row_seq, const int* positions, const int* slot_mapping, float* scores, int cap, float2* stats,
                  int n_head, int n_kv_head, int hd, int ps, float scale, int window, int nsplit) {
  __shared__ float2 sm[DEC_WARPS][16];
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x, hk = blockIdx.y, split = blockIdx.z;
  const int seq = row_seq[row];
  if (seq < 0) return;                       // a padding row of a fixed-size batch
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int pos = positions[row], nq = n_head / n_kv_head, h0 = hk * nq;
  const MixSplit sp = mix_split(pos, window, nsplit);
  const int ks = (sp.kstart & ~15) + split * sp.per, ke = min(sp.kend, ks + sp.per);
  const int* bt = block_table + (size_t)seq * max_blocks;
  if (k_off >= 0 && pos >= ks && pos < ke) {      // uniform over the block: the current key first, the loop reads it like any other
    const int slot = slot_mapping[row];
    if (slot >= 0 && (int)threadIdx.x * 8 < hd)
      *reinterpret_cast<uint4*>(kc + (((size_t)(slot / ps) * n_kv_head + hk) * ps + slot % ps) * hd + threadIdx.x * 8) =
          *reinterpret_cast<const uint4*>(qkv + (size_t)row * ld + k_off + hk * hd + threadIdx.x * 8);
    __syncthreads();
  }
  for (int hb = 0; hb < nq; hb += 16) {           // sixteen query heads at a time: rows g and g + 8 of the A operand
    uint4 qa[2][NC];
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const int h = hb + u * 8 + g, d = c * 32 + t * 8;
        qa[u][c] = h < nq && d < hd ? *reinterpret_cast<const uint4*>(qkv + (size_t)row * ld + (size_t)(h0 + h) * hd + d)
                                    : make_uint4(0, 0, 0, 0);
      }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    uint4 kb[2][NC];
    auto load = [&](int j0) {
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        const int j = j0 + nt * 8 + g;
        const bool in = j < ke;
        const int page = in ? bt[j / ps] : 0;
        const __nv_bfloat16* kp = kc + (((size_t)page * n_kv_head + hk) * ps + (in ? j % ps : 0)) * hd + t * 8;
#pragma unroll
        for (int c = 0; c < NC; ++c)
          kb[nt][c] = in && c * 32 + t * 8 < hd ? ldcg16(kp + c * 32) : make_uint4(0, 0, 0, 0);
      }
    };
    int j0 = ks + warp * 16;
    if (j0 < ke) load(j0);
    for (; j0 < ke; j0 += DEC_WARPS * 16) {
      float sc[2][4];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f;
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          mma_16816(sc[nt], qa[0][c].x, qa[1][c].x, qa[0][c].y, qa[1][c].y, kb[nt][c].x, kb[nt][c].y);
          mma_16816(sc[nt], qa[0][c].z, qa[1][c].z, qa[0][c].w, qa[1][c].w, kb[nt][c].z, kb[nt][c].w);
        }
      }
      if (j0 + DEC_WARPS * 16 < ke) load(j0 + DEC_WARPS * 16);      // the scores above were the last use of these keys
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int h = hb + u * 8 + g;
        if (h >= nq) continue;
        float s[4], mx = m[u];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = j0 + (e >> 1) * 8 + 2 * t + (e & 1);
          const float v = sc[e >> 1][u * 2 + (e & 1)] * scale;
          s[e] = j >= sp.kstart && j < ke ? v : -INFINITY;
          mx = fmaxf(mx, s[e]);
        }
        float* dst = scores + ((size_t)row * n_head + h0 + h) * cap + j0 + 2 * t;
        *reinterpret_cast<float2*>(dst) = make_float2(s[0], s[1]);
        *reinterpret_cast<float2*>(dst + 8) = make_float2(s[2], s[3]);
        if (mx > -INFINITY) {
          float add = 0.f;
#pragma unroll
          for (int e = 0; e < 4; ++e) add += expf(s[e] - mx);
          l[u] = l[u] * expf(m[u] - mx) + add;
          m[u] = mx;
        }
      }
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
#pragma unroll
      for (int o = 1; o < 4; o <<= 1) {
        const float mo = __shfl_xor_sync(0xffffffffu, m[u], o), lo = __shfl_xor_sync(0xffffffffu, l[u], o);
        const float mm = fmaxf(m[u], mo);
        l[u] = mm > -INFINITY ? l[u] * expf(m[u] - mm) + lo * expf(mo - mm) : 0.f;
        m[u] = mm;
      }
      if (t == 0) sm[warp][u * 8 + g] = make_float2(m[u], l[u]);
    }
    __syncthreads();
    if (threadIdx.x < 16 && hb + (int)threadIdx.x < nq) {
      float mm = -INFINITY, ll = 0.f;
#pragma unroll
      for (int w = 0; w < DEC_WARPS; ++w) mm = fmaxf(mm, sm[w][threadIdx.x].x);
#pragma unroll
      for (int w = 0; w < DEC_WARPS; ++w)
        if (sm[w][threadIdx.x].x > -INFINITY) ll += sm[w][threadIdx.x].y * expf(sm[w][threadIdx.x].x - mm);
      stats[((size_t)row * n_head + h0 + hb + threadIdx.x) * nsplit + split] = make_float2(mm, ll);
    }
    __syncthreads();
  }
}

// grid (rows, n_kv_head * pieces of NQ of the heads that share a value head, nsplit).  LPK lanes a value row (8 entries
// each).  Dynamic shared memory: 2 H floats, NQ * H, NQ * MIX_KEYS, DEC_WARPS * NQ * vd.
template <int LPK, int NQ>
__global__ void __launch_bounds__(DEC_WARPS * 32, NQ <= 4 ? 4 : 2)      // four blocks per SM, what the splits are sized for
mix_values_kernel(const __nv_bfloat16* qkv, int ld, int v_off, __nv_bfloat16* vc, const int* block_table, int max_blocks,
                  const int* row_seq, const int* positions, const int* slot_mapping, const float* scores, int cap,
                  const float2* stats, const float* __restrict__ talk, const float* __restrict__ sinks,
                  const __nv_bfloat16* gate, int gate_ld, __nv_bfloat16* __restrict__ out, int out_ld, float* part,
                  unsigned int* counters, int n_head, int n_kv_head, int vd, int ps, int window, int nsplit) {
  extern __shared__ float smem[];
  __shared__ bool is_last;
  float* top = smem;                          // every head's maximum
  float* inv = top + n_head;                  // and one over its denominator
  float* tw = inv + n_head;                   // [NQ][H]: T's rows of this block's heads, times inv
  float* wmix = tw + NQ * n_head;             // [NQ][MIX_KEYS]
  float* red = wmix + NQ * MIX_KEYS;          // [DEC_WARPS][NQ][vd]
  pdl_trigger();
  pdl_wait();
  const int group = n_head / n_kv_head, pieces = (group + NQ - 1) / NQ;
  const int row = blockIdx.x, a = blockIdx.y / pieces, h0 = a * group + (blockIdx.y % pieces) * NQ, split = blockIdx.z;
  const int nq = min(NQ, (a + 1) * group - h0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = row_seq[row];
  if (seq < 0) {
    if (split == 0)
      for (int i = tid; i < nq * vd; i += blockDim.x) out[(size_t)row * out_ld + (size_t)h0 * vd + i] = __float2bfloat16_rn(0.f);
    return;
  }
  const int pos = positions[row];
  const MixSplit sp = mix_split(pos, window, nsplit);
  const int from = sp.kstart & ~15, ks0 = from + split * sp.per, ks = max(ks0, sp.kstart), ke = min(sp.kend, ks0 + sp.per);
  const int* bt = block_table + (size_t)seq * max_blocks;
  if (v_off >= 0 && pos >= ks && pos < ke) {
    const int slot = slot_mapping[row];
    if (slot >= 0 && tid * 8 < vd)
      *reinterpret_cast<uint4*>(vc + (((size_t)(slot / ps) * n_kv_head + a) * ps + slot % ps) * vd + tid * 8) =
          *reinterpret_cast<const uint4*>(qkv + (size_t)row * ld + v_off + a * vd + tid * 8);
  }
  __syncthreads();                            // the current token's value is stored
  constexpr int GW = 32 / LPK, UB = LPK < (NQ > 4 ? 4 : 8) ? LPK : (NQ > 4 ? 4 : 8);
  const int sub = lane % LPK, grp = lane / LPK;
  const bool active = sub * 8 < vd;
  uint4 vn[UB];
  auto fetch = [&](int base, int it0) {       // this lane's pieces of UB of the warp's 32 / GW value rows
#pragma unroll
    for (int i = 0; i < UB; ++i) {
      const int j = base + warp * 32 + (it0 + i) * GW + grp;
      vn[i] = make_uint4(0, 0, 0, 0);
      if (active && j < ke) vn[i] = ldcg16(vc + (((size_t)bt[j / ps] * n_kv_head + a) * ps + j % ps) * vd + sub * 8);
    }
  };
  fetch(ks, 0);                               // on their way while the heads' sums and the first weights are computed
  for (int h = warp; h < n_head; h += DEC_WARPS) {      // a warp a head, a lane a split (32 at most)
    const float2 v = lane < nsplit ? stats[((size_t)row * n_head + h) * nsplit + lane] : make_float2(-INFINITY, 0.f);
    const float sink = sinks ? sinks[h] : -INFINITY;
    const float m = fmaxf(warp_max(v.x), sink);
    const float l = warp_sum(v.x > -INFINITY ? v.y * expf(v.x - m) : 0.f) + (sinks ? expf(sink - m) : 0.f);
    if (lane == 0) {
      top[h] = m;
      inv[h] = 1.f / l;
    }
  }
  __syncthreads();
  for (int i = tid; i < NQ * n_head; i += blockDim.x) {
    const int u = i / n_head, gh = i % n_head;
    tw[i] = u < nq ? talk[(size_t)(h0 + u) * n_head + gh] * inv[gh] : 0.f;
  }
  float acc[NQ][8];
#pragma unroll
  for (int u = 0; u < NQ; ++u)
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[u][i] = 0.f;
  for (int base = ks; base < ke; base += MIX_KEYS) {
    __syncthreads();                          // tw is there; wmix of the keys before has been read
    {
      float w[NQ];
#pragma unroll
      for (int u = 0; u < NQ; ++u) w[u] = 0.f;
      if (base + tid < ke) {
        const float* s = scores + (size_t)row * n_head * cap + base + tid;
#pragma unroll 8
        for (int gh = 0; gh < n_head; ++gh) {      // eight scores in flight
          const float e = expf(s[(size_t)gh * cap] - top[gh]);
#pragma unroll
          for (int u = 0; u < NQ; ++u) w[u] = fmaf(tw[u * n_head + gh], e, w[u]);
        }
      }
#pragma unroll
      for (int u = 0; u < NQ; ++u) wmix[u * MIX_KEYS + tid] = w[u];
    }
    __syncthreads();
#pragma unroll
    for (int it0 = 0; it0 < LPK; it0 += UB) {
      uint4 v[UB];
#pragma unroll
      for (int i = 0; i < UB; ++i) v[i] = vn[i];
      if (it0 + UB < LPK) fetch(base, it0 + UB);
      else if (base + MIX_KEYS < ke) fetch(base + MIX_KEYS, 0);
#pragma unroll
      for (int i = 0; i < UB; ++i) {
        float f[8];
        unpack8(v[i], f);
        const int k = warp * 32 + (it0 + i) * GW + grp;
#pragma unroll
        for (int u = 0; u < NQ; ++u) {
          const float w = wmix[u * MIX_KEYS + k];
#pragma unroll
          for (int d = 0; d < 8; ++d) acc[u][d] = fmaf(w, f[d], acc[u][d]);
        }
      }
    }
  }
#pragma unroll
  for (int o = LPK; o < 32; o <<= 1)
#pragma unroll
    for (int u = 0; u < NQ; ++u)
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[u][i] += __shfl_xor_sync(0xffffffffu, acc[u][i], o);
  if (grp == 0 && active) {
#pragma unroll
    for (int u = 0; u < NQ; ++u)
#pragma unroll
      for (int i = 0; i < 8; ++i) red[(warp * NQ + u) * vd + sub * 8 + i] = acc[u][i];
  }
  __syncthreads();
  auto store = [&](int i, float v) {
    const size_t c = (size_t)h0 * vd + i;
    if (gate) v *= sigmoid_f32(to_f32(gate[(size_t)row * gate_ld + c]));
    out[(size_t)row * out_ld + c] = __float2bfloat16_rn(v);
  };
  float* mine = part + (((size_t)row * n_head + h0) * nsplit) * vd;      // [heads of the block][nsplit][vd]
  for (int i = tid; i < nq * vd; i += blockDim.x) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < DEC_WARPS; ++w) v += red[w * NQ * vd + i];
    if (nsplit == 1) store(i, v);
    else mine[((size_t)(i / vd) * nsplit + split) * vd + i % vd] = v;
  }
  if (nsplit == 1) return;
  // the block of this row and these heads that finishes last adds the splits up (and sets the counter back to zero)
  __threadfence();
  __syncthreads();
  unsigned int* counter = counters + (size_t)row * gridDim.y + blockIdx.y;
  if (tid == 0) is_last = atomicAdd(counter, 1u) == (unsigned)nsplit - 1;
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  for (int i = tid * 4; i < nq * vd; i += blockDim.x * 4) {
    const float4* src = reinterpret_cast<const float4*>(mine + (size_t)(i / vd) * nsplit * vd + i % vd);
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < nsplit; ++s) {         // eight loads in flight, added in their order
      const float4 p = __ldcg(src + (size_t)s * (vd / 4));
      v.x += p.x;
      v.y += p.y;
      v.z += p.z;
      v.w += p.w;
    }
    store(i, v.x);
    store(i + 1, v.y);
    store(i + 2, v.z);
    store(i + 3, v.w);
  }
  if (tid == 0) *counter = 0;
}

static int mix_heads_per_block(int group) { return group <= 1 ? 1 : (group <= 2 ? 2 : (group <= 4 ? 4 : 8)); }

}  // namespace cbis

using namespace cbis;

// Blocks of mix_values per row and split (the counters a row needs).
CBIS_EXPORT int cbis_decode_mix_blocks(int n_head, int n_kv_head) {
  const int group = n_head / n_kv_head, nq = mix_heads_per_block(group);
  return n_kv_head * ((group + nq - 1) / nq);
}

// Floats of scratch for `rows` rows: every head's scores of up to `cap` keys (a multiple of 16), the splits' maxima and
// sums, and their partial results.
CBIS_EXPORT long long cbis_decode_mix_scratch_floats(int rows, int n_head, int vd, int cap, int nsplit) {
  return (long long)rows * n_head * cap + (long long)rows * n_head * nsplit * (2 + (nsplit > 1 ? vd : 0)) + 2;
}

// qkv: this step's projections [rows, ld], queries at column 0; k_off / v_off >= 0: the current token's key / value are
// taken from qkv and stored at slot_mapping[row].  talk: [n_head, n_head]; sinks (may be null): [n_head]; gate (may be null):
// [rows, gate_ld].  No request of the step may hold more than cap keys.
CBIS_EXPORT int cbis_decode_mix_bf16(const void* qkv, int ld, int k_off, int v_off, void* kc, void* vc,
                                     const int* block_table, int max_blocks, const int* row_seq, const int* positions,
                                     const int* slot_mapping, const float* talk, const float* sinks, const void* gate,
                                     int gate_ld, void* out, int out_ld, float* scratch, unsigned int* counters, int cap,
                                     int rows, int n_head, int n_kv_head, int hd, int vd, int ps, float scale, int window,
                                     int nsplit, void* stream) {
  if (rows <= 0) return CBIS_OK;
  if (hd <= 0 || hd > 256 || hd % 8 || vd <= 0 || vd > 256 || vd % 8 || ps <= 0 || n_head <= 0 || n_kv_head <= 0 ||
      n_head % n_kv_head || n_head > 128 || nsplit < 1 || nsplit > 32 || cap <= 0 || cap % 16 || !scratch || !talk ||
      (nsplit > 1 && !counters))
    return CBIS_ERR_BAD_SIZE;
  if (ld % 8 || (k_off >= 0 && k_off % 8) || (v_off >= 0 && v_off % 8) ||
      (((uintptr_t)qkv | (uintptr_t)kc | (uintptr_t)vc | (uintptr_t)scratch) & 15))
    return CBIS_ERR_ALIGNMENT;
  cudaStream_t st = (cudaStream_t)stream;
  float* scores = scratch;
  float2* stats = reinterpret_cast<float2*>(scores + (size_t)rows * n_head * cap);
  float* part = reinterpret_cast<float*>(stats + (((size_t)rows * n_head * nsplit + 1) & ~(size_t)1));      // 16-byte aligned
  typedef __nv_bfloat16 bf;
  cudaError_t e = cudaErrorInvalidValue;
#define CBIS_SC(NC)                                                                                                   \
  e = launch_pdl(mix_scores_kernel<NC>, dim3(rows, n_kv_head, nsplit), dim3(DEC_WARPS * 32), 0, st, (const bf*)qkv, ld, k_off, \
                 (bf*)kc, block_table, max_blocks, row_seq, positions, slot_mapping, scores, cap, stats, n_head, n_kv_head, \
                 hd, ps, scale, window, nsplit)
  const int nc = (hd + 31) / 32;
  if (nc <= 1) CBIS_SC(1);
  else if (nc == 2) CBIS_SC(2);
  else if (nc == 3) CBIS_SC(3);
  else if (nc == 4) CBIS_SC(4);
  else if (nc <= 6) CBIS_SC(6);
  else CBIS_SC(8);
#undef CBIS_SC
  if (e != cudaSuccess) return (int)e;
  const int nq = mix_heads_per_block(n_head / n_kv_head);
  const size_t smem = ((size_t)2 * n_head + (size_t)nq * n_head + (size_t)nq * MIX_KEYS + (size_t)DEC_WARPS * nq * vd) * sizeof(float);
  const dim3 grid(rows, cbis_decode_mix_blocks(n_head, n_kv_head), nsplit);
#define CBIS_VA(LPK, NQ)                                                                                              \
  do {                                                                                                                \
    e = launch_pdl(mix_values_kernel<LPK, NQ>, grid, dim3(DEC_WARPS * 32), smem, st, (const bf*)qkv, ld, v_off, (bf*)vc, \
                   block_table, max_blocks, row_seq, positions, slot_mapping, (const float*)scores, cap,              \
                   (const float2*)stats, talk, sinks, (const bf*)gate, gate_ld, (bf*)out, out_ld, part, counters,     \
                   n_head, n_kv_head, vd, ps, window, nsplit);                                                        \
  } while (0)
#define CBIS_VA_NQ(LPK)                                                                                               \
  do {                                                                                                                \
    if (nq == 1) CBIS_VA(LPK, 1);                                                                                     \
    else if (nq == 2) CBIS_VA(LPK, 2);                                                                                \
    else if (nq == 4) CBIS_VA(LPK, 4);                                                                                \
    else CBIS_VA(LPK, 8);                                                                                             \
  } while (0)
  if (vd <= 32) CBIS_VA_NQ(4);
  else if (vd <= 64) CBIS_VA_NQ(8);
  else if (vd <= 128) CBIS_VA_NQ(16);
  else CBIS_VA_NQ(32);
#undef CBIS_VA_NQ
#undef CBIS_VA
  return (int)e;
}
