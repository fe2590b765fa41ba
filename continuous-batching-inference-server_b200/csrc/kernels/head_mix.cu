// Around attention whose heads share more than keys and values, in 32-bit arithmetic whatever the storage type.
//
//   qk_head_norm: every head of q and of k (columns of a projection, in place) is divided by its own root mean square and
//   multiplied by a weight as wide as ONE head, shared by all heads of q, another shared by all heads of k.
//
//   mix_heads: attention whose softmax weights are mixed across heads before they meet the values,
//     w'_h = sum_g T[h, g] w_g,   out_h = w'_h V_{kv(h)},   kv(h) = h / (H / G).
//   The sum over the keys and the sum over the heads may be taken in either order: with o[g, a] = w_g V_a (every query head
//   over the values of every key/value head a),
//     out_h = sum_g T[h, g] o[g, kv(h)],
//   which this kernel takes, with an optional gate on the result, element by element: out_h * sigmoid(gate_h).
#include "common.cuh"

namespace cbis {

template <typename TT, int V>
struct alignas(sizeof(TT) * V) Pack {
  TT e[V];
};

// A warp per (row, head); a lane holds up to NV packs of V entries.  In place.
template <typename TT, int V, int NV>
__global__ void __launch_bounds__(256)
qk_head_norm_kernel(TT* buf, int ld, int q_off, int q_heads, int k_off, int k_heads, int width,
                    const float* __restrict__ q_w, const float* __restrict__ k_w, float eps, int rows) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, heads = q_heads + k_heads;
  const long long unit = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (unit >= (long long)rows * heads) return;
  const int r = (int)(unit / heads), h = (int)(unit % heads);
  const bool is_q = h < q_heads;
  TT* b = buf + (size_t)r * ld + (is_q ? q_off + h * width : k_off + (h - q_heads) * width);
  const float* w = is_q ? q_w : k_w;
  float v[NV][V], ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * 32 + lane) * V;
    Pack<TT, V> p;
    const bool in = c < width;
    if (in) p = *reinterpret_cast<const Pack<TT, V>*>(b + c);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      v[i][k] = in ? to_f32(p.e[k]) : 0.f;
      ss = fmaf(v[i][k], v[i][k], ss);
    }
  }
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)width + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * 32 + lane) * V;
    if (c < width) {
      Pack<TT, V> p;
#pragma unroll
      for (int k = 0; k < V; ++k) from_f32(p.e[k], v[i][k] * inv * w[c + k]);
      *reinterpret_cast<Pack<TT, V>*>(b + c) = p;
    }
  }
}

// grid (rows, pieces of the G * vd / V packs); shared: H * H floats (T).  o: [rows, H * G * vd], head g's part over value
// head a at column (g * G + a) * vd.  A thread takes one pack of one value head for all the heads h that read it, HG of
// them at a time (their sums in registers), so o is read once where H / G <= HG.
template <typename TT, int V, int HG>
__global__ void __launch_bounds__(128)
mix_heads_kernel(const TT* o, int o_ld, const float* __restrict__ talk, const TT* gate, int gate_ld, TT* out, int out_ld,
                 int H, int G, int vd) {
  extern __shared__ float t[];
  pdl_trigger();
  for (int i = threadIdx.x; i < H * H; i += blockDim.x) t[i] = talk[i];
  pdl_wait();
  __syncthreads();
  const int r = blockIdx.x, per_head = vd / V, unit = blockIdx.y * blockDim.x + threadIdx.x, group = H / G;
  if (unit >= G * per_head) return;
  const int a = unit / per_head, d = (unit % per_head) * V;
  const TT* src = o + (size_t)r * o_ld + a * vd + d;
  for (int h0 = a * group; h0 < (a + 1) * group; h0 += HG) {
    float acc[HG][V];
#pragma unroll
    for (int u = 0; u < HG; ++u)
#pragma unroll
      for (int k = 0; k < V; ++k) acc[u][k] = 0.f;
    const int n = min(HG, (a + 1) * group - h0);
#pragma unroll 8
    for (int g = 0; g < H; ++g) {      // eight loads in flight
      const Pack<TT, V> p = *reinterpret_cast<const Pack<TT, V>*>(src + (size_t)g * G * vd);
#pragma unroll
      for (int u = 0; u < HG; ++u) {
        if (u < n) {
          const float f = t[(h0 + u) * H + g];
#pragma unroll
          for (int k = 0; k < V; ++k) acc[u][k] = fmaf(f, to_f32(p.e[k]), acc[u][k]);
        }
      }
    }
#pragma unroll
    for (int u = 0; u < HG; ++u) {
      if (u < n) {
        const size_t c = (size_t)(h0 + u) * vd + d;
        Pack<TT, V> p, q;
        if (gate) q = *reinterpret_cast<const Pack<TT, V>*>(gate + (size_t)r * gate_ld + c);
#pragma unroll
        for (int k = 0; k < V; ++k) from_f32(p.e[k], gate ? acc[u][k] * sigmoid_f32(to_f32(q.e[k])) : acc[u][k]);
        *reinterpret_cast<Pack<TT, V>*>(out + (size_t)r * out_ld + c) = p;
      }
    }
  }
}

}  // namespace cbis

using namespace cbis;

CBIS_EXPORT int cbis_mix_heads_max_heads() { return 224; }      // H * H floats of shared memory

// buf [rows, ld] of the compute type, changed in place: q at columns q_off.. (q_heads x width), k at k_off.. (k_heads x
// width; k_heads 0: none).  q_w, k_w: `width` numbers each.
CBIS_EXPORT int cbis_qk_head_norm(void* buf, int ld, int q_off, int q_heads, int k_off, int k_heads, int width,
                                  const float* q_w, const float* k_w, float eps, int rows, int dtype, void* stream) {
  if (rows <= 0 || q_heads + k_heads <= 0) return CBIS_OK;
  if (q_heads < 0 || k_heads < 0 || width <= 0 || width > 512 || (q_heads && !q_w) || (k_heads && !k_w)) return CBIS_ERR_BAD_SIZE;
  const long long units = (long long)rows * (q_heads + k_heads);
  const dim3 grid((unsigned)((units + 7) / 8));
  cudaStream_t st = (cudaStream_t)stream;
  const int esz = dtype == CBIS_F32 ? 4 : 2;
  const bool vec = width % 4 == 0 && ld % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && !((uintptr_t)buf & (4 * esz - 1));
#define CBIS_QKH(TT, V, NV)                                                                                          \
  return (int)launch_pdl(qk_head_norm_kernel<TT, V, NV>, grid, dim3(256), 0, st, (TT*)buf, ld, q_off, q_heads, k_off, \
                         k_heads, width, q_w, k_w, eps, rows)
#define CBIS_QKH_PICK(TT)                   \
  do {                                      \
    if (vec && width <= 128) CBIS_QKH(TT, 4, 1); \
    if (vec) CBIS_QKH(TT, 4, 4);            \
    CBIS_QKH(TT, 1, 16);                    \
  } while (0)
  if (dtype == CBIS_F32) CBIS_QKH_PICK(float);
  if (dtype == CBIS_BF16) CBIS_QKH_PICK(__nv_bfloat16);
#undef CBIS_QKH_PICK
#undef CBIS_QKH
  return CBIS_ERR_BAD_DTYPE;
}

// talk: [H, H] 32-bit; gate (may be null): [rows, gate_ld], H * vd columns; out: [rows, H * vd].
CBIS_EXPORT int cbis_mix_heads(const void* o, int o_ld, const float* talk, const void* gate, int gate_ld, void* out,
                               int out_ld, int rows, int H, int G, int vd, int dtype, void* stream) {
  if (rows <= 0) return CBIS_OK;
  if (H <= 0 || G <= 0 || H % G || vd <= 0) return CBIS_ERR_BAD_SIZE;
  if (H > cbis_mix_heads_max_heads()) return CBIS_ERR_TOO_LARGE;
  cudaStream_t st = (cudaStream_t)stream;
  const int esz = dtype == CBIS_F32 ? 4 : 2;
  const bool vec = vd % 4 == 0 && o_ld % 4 == 0 && out_ld % 4 == 0 && (!gate || gate_ld % 4 == 0) &&
                   !(((uintptr_t)o | (uintptr_t)out | (uintptr_t)gate) & (4 * esz - 1));
  const size_t smem = (size_t)H * H * sizeof(float);
  const int packs = G * (vd / (vec ? 4 : 1)), threads = packs >= 128 ? 128 : (packs >= 64 ? 64 : 32);
  const dim3 grid(rows, (packs + threads - 1) / threads);
#define CBIS_MIX(TT, V)                                                                                              \
  do {                                                                                                               \
    if (smem > 48 * 1024) {                                                                                          \
      const cudaError_t e = cudaFuncSetAttribute(mix_heads_kernel<TT, V, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (e != cudaSuccess) return (int)e;                                                                           \
    }                                                                                                                \
    return (int)launch_pdl(mix_heads_kernel<TT, V, 4>, grid, dim3(threads), smem, st, (const TT*)o, o_ld, talk,      \
                           (const TT*)gate, gate_ld, (TT*)out, out_ld, H, G, vd);                                    \
  } while (0)
  if (dtype == CBIS_F32) {
    if (vec) CBIS_MIX(float, 4);
    CBIS_MIX(float, 1);
  }
  if (dtype == CBIS_BF16) {
    if (vec) CBIS_MIX(__nv_bfloat16, 4);
    CBIS_MIX(__nv_bfloat16, 1);
  }
#undef CBIS_MIX
  return CBIS_ERR_BAD_DTYPE;
}
