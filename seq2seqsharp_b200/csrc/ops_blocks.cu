// Building blocks of layered engines (engine_layers.cuh) around their linears and attention:
//   block_norm_kernel    pending expert outputs -> residual, RMS norm in groups with one or two weights from one pass over the
//                        row, the second result optionally also in the row order of a grouped product, and for one new
//                        position per sequence the short causal convolution with its state;
//   sandwich_norm_kernel the sublayer output's own norm and scale -> residual, norm of the sum for the next sublayer, one pass;
//   short_conv_kernel    the same convolution for many new positions; short_conv_state_kernel then leaves the sequence's last
//                        inputs in its ring (a kernel of its own: the ring is read by the first positions of a portion);
//   table_route_kernel   experts chosen by token id: for every layer the picks of all rows sorted by expert, cut into blocks of
//                        rows of one expert (the unit of the grouped products), all layers in one launch at the start of a step;
//   pick_linear_kernel   one row times its own expert's matrix on CUDA cores: fp32 models and shapes the grouped
//                        tensor-core products do not take.
// Convolution state: a ring of `taps` rows per sequence, position p at row p % taps.  With one row more than the convolution looks
// back, a step that is run again at the same position (a sequence that stands still while others go on) finds the ring as it was.
#include "kernels.cuh"

namespace tsb {

TSB_CHECKED_WORD(blocks)
#ifndef TSB200_CHECKED
int chk_take_blocks() { return 0; }
#endif

template <typename T, int V> struct VecIO;   // V consecutive elements
template <typename T> struct VecIO<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float* f) { f[0] = to_f<T>(p[0]); }
  static __device__ __forceinline__ void store(T* p, const float* f) { p[0] = from_f<T>(f[0]); }
};
template <> struct VecIO<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float* f) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    f[0] = t.x; f[1] = t.y; f[2] = t.z; f[3] = t.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};
template <> struct VecIO<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* f) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = Pair16<__nv_bfloat16>::get(t.x), b = Pair16<__nv_bfloat16>::get(t.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* f) {
    *reinterpret_cast<uint2*>(p) = make_uint2(Pair16<__nv_bfloat16>::put(f[0], f[1]), Pair16<__nv_bfloat16>::put(f[2], f[3]));
  }
};

constexpr int kBlockNormThreads = 256;

// shared memory: the row in fp32 [d], partial sums [max(groups, 8)]
template <typename T, int V>
__global__ void __launch_bounds__(kBlockNormThreads) block_norm_kernel(BlockNormArgs a) {
  extern __shared__ float s_row[];
  float* s_part = s_row + a.d;
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
  const int d = a.d, gsz = d / a.groups;
  const int out_row = blockIdx.x;
  int row = out_row;
  if (a.rows_of) row = a.rows_of[out_row];
  else if (a.last_of_S > 0) {
    const int n = a.lens ? a.lens[out_row] : a.last_of_S;
    row = out_row * a.last_of_S + min(max(n, 1), a.last_of_S) - 1;
  }
  float* xr = a.x + (int64_t)row * d;
  const float inv_top = a.top > 0 ? 1.0f / (float)a.top : 0.0f;
  for (int i = tid * V; i < d; i += kBlockNormThreads * V) {
    float v[V];
    VecIO<float, V>::load(xr + i, v);
    if (a.y) {   // the previous layer's experts: their mean, gated, joins the residual here
      float sum[V];
#pragma unroll
      for (int e = 0; e < V; ++e) sum[e] = 0.0f;
      for (int j = 0; j < a.top; ++j) {
        float t[V];
        VecIO<T, V>::load(reinterpret_cast<const T*>(a.y) + (int64_t)a.y_pos[(int64_t)row * a.top + j] * d + i, t);
#pragma unroll
        for (int e = 0; e < V; ++e) sum[e] += t[e];
      }
      float g[V];
      if (a.y_gate) VecIO<T, V>::load(reinterpret_cast<const T*>(a.y_gate) + (int64_t)row * d + i, g);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += sum[e] * inv_top * (a.y_gate ? g[e] : 1.0f);
      if (a.write_x) VecIO<float, V>::store(xr + i, v);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) s_row[i + e] = v[e];
  }
  __syncthreads();
  // sums of squares: several warps per group when there are few groups, several groups per warp otherwise
  const int wpg = a.groups >= 8 ? 1 : 8 / a.groups;
  if (a.groups >= 8) {
    for (int g = w; g < a.groups; g += 8) {
      float s = 0.0f;
      for (int i = lane; i < gsz; i += 32) s += s_row[g * gsz + i] * s_row[g * gsz + i];
      s = warp_sum(s);
      if (lane == 0) s_part[g] = s;
    }
  } else {
    const int g = w / wpg, part = w % wpg;
    float s = 0.0f;
    if (g < a.groups)
      for (int i = part * 32 + lane; i < gsz; i += wpg * 32) s += s_row[g * gsz + i] * s_row[g * gsz + i];
    s = warp_sum(s);
    if (lane == 0) s_part[w] = s;
  }
  __syncthreads();
  auto inv_rms = [&](int g) {
    float s = 0.0f;
    for (int q = 0; q < wpg; ++q) s += s_part[g * wpg + q];
    return 1.0f / sqrtf(s / (float)gsz + a.eps);
  };
  int b = 0, pos = 0;
  if (a.conv_ring) {
    b = out_row;
    pos = state_len(a.state, b, a.T0);
  }
  int cur_g = -1;
  float inv = 0.0f;
  for (int i = tid * V; i < d; i += kBlockNormThreads * V) {
    float n[V], h[V], wt[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const int g = (i + e) / gsz;
      if (g != cur_g) {
        cur_g = g;
        inv = inv_rms(g);
      }
      n[e] = s_row[i + e] * inv;
    }
    VecIO<T, V>::load(reinterpret_cast<const T*>(a.w1) + i, wt);
#pragma unroll
    for (int e = 0; e < V; ++e) h[e] = n[e] * wt[e] * a.out_scale;
    VecIO<T, V>::store(reinterpret_cast<T*>(a.h1) + (int64_t)out_row * d + i, h);
    if (a.w2) {
      float h2[V];
      VecIO<T, V>::load(reinterpret_cast<const T*>(a.w2) + i, wt);
#pragma unroll
      for (int e = 0; e < V; ++e) h2[e] = n[e] * wt[e];
      VecIO<T, V>::store(reinterpret_cast<T*>(a.h2) + (int64_t)out_row * d + i, h2);
      for (int j = 0; j < a.next_top; ++j)
        VecIO<T, V>::store(reinterpret_cast<T*>(a.h2_sorted) + (int64_t)a.next_pos[(int64_t)row * a.next_top + j] * d + i, h2);
    }
    if (a.conv_ring) {
      T* ring = reinterpret_cast<T*>(a.conv_ring) + (int64_t)b * a.taps * d;
      float out[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float hr = to_f<T>(from_f<T>(h[e]));   // the value the state keeps
        float acc = hr;
        const T* cw = reinterpret_cast<const T*>(a.conv_w) + (int64_t)(i + e) * a.taps;
        for (int j = 0; j < a.taps; ++j) {
          const int p = pos - a.taps + 1 + j;
          if (p < 0) continue;
          acc += to_f<T>(cw[j]) * (p == pos ? hr : to_f<T>(ring[(int64_t)(p % a.taps) * d + i + e]));
        }
        out[e] = acc;
      }
      VecIO<T, V>::store(ring + (int64_t)(pos % a.taps) * d + i, h);
      VecIO<T, V>::store(reinterpret_cast<T*>(a.hc) + (int64_t)out_row * d + i, out);
    }
  }
}

// The same for the usual widths, the row in registers: thread t holds elements (t + u * threads) * 4 .. + 3.  Weights are requested
// before the wait on the previous kernel, everything that depends on it in one round afterwards.  Groups are 2^k * 4 elements inside a
// warp's 128, or whole multiples of 128.  TAPS: room for the convolution's taps, 0: none.
constexpr int kFastTop = 8;
template <typename T, int NV, int TAPS>
__global__ void __launch_bounds__(512) block_norm_fast_kernel(BlockNormArgs a) {
  __shared__ float s_part[16 * NV];
  pdl_trigger();
  const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, w = tid >> 5, nw = nt >> 5;
  const int d = a.d, gsz = d / a.groups, out_row = blockIdx.x;
  float w1[NV][4], w2[NV][4], cw[NV][4][TAPS > 0 ? TAPS : 1];
#pragma unroll
  for (int u = 0; u < NV; ++u) {
    const int i = (tid + u * nt) * 4;
    VecIO<T, 4>::load(reinterpret_cast<const T*>(a.w1) + i, w1[u]);
    if (a.w2) VecIO<T, 4>::load(reinterpret_cast<const T*>(a.w2) + i, w2[u]);
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int e = 0; e < 4; ++e)
#pragma unroll
        for (int q = 0; q < TAPS; ++q)   // q positions back
          cw[u][e][q] = q < a.taps ? to_f<T>(reinterpret_cast<const T*>(a.conv_w)[(int64_t)(i + e) * a.taps + a.taps - 1 - q]) : 0.0f;
    }
  }
  pdl_wait();
  int row = out_row;
  if (a.rows_of) row = a.rows_of[out_row];
  else if (a.last_of_S > 0) {
    const int n = a.lens ? a.lens[out_row] : a.last_of_S;
    row = out_row * a.last_of_S + min(max(n, 1), a.last_of_S) - 1;
  }
  float* xr = a.x + (int64_t)row * d;
  int yp[kFastTop], np[kFastTop];
#pragma unroll
  for (int j = 0; j < kFastTop; ++j) {
    yp[j] = a.y && j < a.top ? a.y_pos[(int64_t)row * a.top + j] : 0;
    np[j] = a.w2 && j < a.next_top ? a.next_pos[(int64_t)row * a.next_top + j] : 0;
  }
  float v[NV][4], past[NV][TAPS > 1 ? TAPS - 1 : 1][4];
  int pos = 0;
  T* ring = nullptr;
  if constexpr (TAPS > 0) {
    pos = state_len(a.state, out_row, a.T0);
    ring = reinterpret_cast<T*>(a.conv_ring) + (int64_t)out_row * a.taps * d;
  }
#pragma unroll
  for (int u = 0; u < NV; ++u) {
    const int i = (tid + u * nt) * 4;
    VecIO<float, 4>::load(xr + i, v[u]);
    if constexpr (TAPS > 1) {
#pragma unroll
      for (int q = 1; q < TAPS; ++q) {
        if (q < a.taps && pos >= q) VecIO<T, 4>::load(ring + (int64_t)((pos - q) % a.taps) * d + i, past[u][q - 1]);
        else past[u][q - 1][0] = past[u][q - 1][1] = past[u][q - 1][2] = past[u][q - 1][3] = 0.0f;
      }
    }
  }
  if (a.y) {
    const float inv_top = 1.0f / (float)a.top;
#pragma unroll
    for (int u = 0; u < NV; ++u) {
      const int i = (tid + u * nt) * 4;
      float g[4] = {1.0f, 1.0f, 1.0f, 1.0f}, sum[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      if (a.y_gate) VecIO<T, 4>::load(reinterpret_cast<const T*>(a.y_gate) + (int64_t)row * d + i, g);
#pragma unroll
      for (int j = 0; j < kFastTop; ++j)
        if (j < a.top) {
          float t[4];
          VecIO<T, 4>::load(reinterpret_cast<const T*>(a.y) + (int64_t)yp[j] * d + i, t);
#pragma unroll
          for (int e = 0; e < 4; ++e) sum[e] += t[e];
        }
#pragma unroll
      for (int e = 0; e < 4; ++e) v[u][e] += sum[e] * inv_top * g[e];
      if (a.write_x) VecIO<float, 4>::store(xr + i, v[u]);
    }
  }
  float inv[NV];
#pragma unroll
  for (int u = 0; u < NV; ++u) {
    float s = (v[u][0] * v[u][0] + v[u][1] * v[u][1]) + (v[u][2] * v[u][2] + v[u][3] * v[u][3]);
    if (gsz < 128) {
      for (int o = gsz >> 3; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    } else {
      s = warp_sum(s);
      if (lane == 0) s_part[w + u * nw] = s;
    }
    inv[u] = s;
  }
  if (gsz >= 128) {
    __syncthreads();
    const int per = gsz >> 7;
#pragma unroll
    for (int u = 0; u < NV; ++u) {
      const int first = (w + u * nw) / per * per;
      float s = 0.0f;
      for (int q = 0; q < per; ++q) s += s_part[first + q];
      inv[u] = s;
    }
  }
#pragma unroll
  for (int u = 0; u < NV; ++u) {
    const int i = (tid + u * nt) * 4;
    const float r = 1.0f / sqrtf(inv[u] / (float)gsz + a.eps);
    float h[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) h[e] = v[u][e] * r * w1[u][e] * a.out_scale;
    VecIO<T, 4>::store(reinterpret_cast<T*>(a.h1) + (int64_t)out_row * d + i, h);
    if (a.w2) {
      float h2[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) h2[e] = v[u][e] * r * w2[u][e];
      VecIO<T, 4>::store(reinterpret_cast<T*>(a.h2) + (int64_t)out_row * d + i, h2);
#pragma unroll
      for (int j = 0; j < kFastTop; ++j)
        if (j < a.next_top) VecIO<T, 4>::store(reinterpret_cast<T*>(a.h2_sorted) + (int64_t)np[j] * d + i, h2);
    }
    if constexpr (TAPS > 0) {
      float out[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float hr = to_f<T>(from_f<T>(h[e]));   // the value the state keeps
        float acc = hr;
#pragma unroll
        for (int q = TAPS - 1; q >= 1; --q) acc += cw[u][e][q] * past[u][q - 1][e];   // oldest first, as in the other kernels
        out[e] = acc + cw[u][e][0] * hr;
      }
      VecIO<T, 4>::store(ring + (int64_t)(pos % a.taps) * d + i, h);
      VecIO<T, 4>::store(reinterpret_cast<T*>(a.hc) + (int64_t)out_row * d + i, out);
    }
  }
}
static bool block_norm_fast_shape(const BlockNormArgs& a) {
  const int gsz = a.d / a.groups, nv = a.d <= 2048 ? 1 : 2;
  if (a.d % (128 * nv) != 0 || a.d > 4096 || a.top > kFastTop || a.next_top > kFastTop || (a.conv_ring && a.taps > 4)) return false;
  return gsz >= 128 ? gsz % 128 == 0 : (gsz >= 4 && (gsz & (gsz - 1)) == 0);
}

// Both norms of a sandwich block in one pass: the row of x and of the sublayer output y in registers (thread t holds elements
// (t + u * threads) * V .. + V - 1), weights requested before the wait on the previous kernel.
__device__ __forceinline__ float sandwich_sum(float v, float* red) {   // block-wide sum, one barrier; red: 32 floats of its own per call
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
  v = warp_sum(v);
  if (lane == 0) red[w] = v;
  __syncthreads();
  return warp_sum(lane < nw ? red[lane] : 0.0f);
}
template <typename T, int V, int NV>
__global__ void __launch_bounds__(512) sandwich_norm_kernel(SandwichNormArgs a) {
  __shared__ float s_red[2][32];
  pdl_trigger();
  const int tid = threadIdx.x, nt = blockDim.x, d = a.d, out_row = blockIdx.x;
  constexpr bool kEarly = NV <= 2;   // room to hold the weights across the wait
  float pw[kEarly ? NV : 1][V], nw[kEarly ? NV : 1][V];
  auto post_weight = [&](int i, float* o) {
    VecIO<T, V>::load(reinterpret_cast<const T*>(a.post_w) + i, o);
    if (a.scale) {
      float sc[V];
      VecIO<T, V>::load(reinterpret_cast<const T*>(a.scale) + i, sc);
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] *= sc[e];
    }
  };
  if constexpr (kEarly) {
#pragma unroll
    for (int u = 0; u < NV; ++u) {
      const int i = (tid + u * nt) * V;
      if (i < d) {
        if (a.y) post_weight(i, pw[u]);
        VecIO<T, V>::load(reinterpret_cast<const T*>(a.next_w) + i, nw[u]);
      }
    }
  }
  pdl_wait();
  int row = out_row;
  if (a.rows_of) row = a.rows_of[out_row];
  else if (a.last_of_S > 0) {
    const int n = a.lens ? a.lens[out_row] : a.last_of_S;
    row = out_row * a.last_of_S + min(max(n, 1), a.last_of_S) - 1;
  }
  float* xr = a.x + (int64_t)row * d;
  float x[NV][V];
#pragma unroll
  for (int u = 0; u < NV; ++u) {
    const int i = (tid + u * nt) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) x[u][e] = 0.0f;
    if (i < d) VecIO<float, V>::load(xr + i, x[u]);
  }
  if (a.y) {
    const T* yr = reinterpret_cast<const T*>(a.y) + (int64_t)row * d;
    float y[NV][V], s = 0.0f;
#pragma unroll
    for (int u = 0; u < NV; ++u) {
      const int i = (tid + u * nt) * V;
#pragma unroll
      for (int e = 0; e < V; ++e) y[u][e] = 0.0f;
      if (i < d) VecIO<T, V>::load(yr + i, y[u]);
#pragma unroll
      for (int e = 0; e < V; ++e) s += y[u][e] * y[u][e];
    }
    const float r = 1.0f / sqrtf(sandwich_sum(s, s_red[0]) / (float)d + a.eps);
#pragma unroll
    for (int u = 0; u < NV; ++u) {
      const int i = (tid + u * nt) * V;
      if (i < d) {
        float w[V];
        if constexpr (!kEarly) post_weight(i, w);
#pragma unroll
        for (int e = 0; e < V; ++e) x[u][e] += y[u][e] * r * (kEarly ? pw[kEarly ? u : 0][e] : w[e]);
        if (a.write_x) VecIO<float, V>::store(xr + i, x[u]);
      }
    }
  }
  float s = 0.0f;
#pragma unroll
  for (int u = 0; u < NV; ++u)
#pragma unroll
    for (int e = 0; e < V; ++e) s += x[u][e] * x[u][e];
  const float r = 1.0f / sqrtf(sandwich_sum(s, s_red[1]) / (float)d + a.eps);
#pragma unroll
  for (int u = 0; u < NV; ++u) {
    const int i = (tid + u * nt) * V;
    if (i < d) {
      float w[V], h[V];
      if constexpr (!kEarly) VecIO<T, V>::load(reinterpret_cast<const T*>(a.next_w) + i, w);
#pragma unroll
      for (int e = 0; e < V; ++e) h[e] = x[u][e] * r * (kEarly ? nw[kEarly ? u : 0][e] : w[e]);
      VecIO<T, V>::store(reinterpret_cast<T*>(a.h) + (int64_t)out_row * d + i, h);
    }
  }
}

// out[b, s] = h[b, s] + sum_j w[:, j] h[b, s - taps + 1 + j]; positions before the portion come from the ring, none before 0
template <typename T>
__global__ void __launch_bounds__(256) short_conv_kernel(T* out, const T* h, const T* wgt, const T* ring, int B, int S, int d, int taps, int T0_arg,
                                                         const int* state) {
  const int64_t n = (int64_t)B * S * d;
  for (int64_t q = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; q < n; q += (int64_t)gridDim.x * blockDim.x) {
    const int i = (int)(q % d);
    const int64_t row = q / d;
    const int b = (int)(row / S), s = (int)(row % S);
    const int T0 = state_len(state, b, T0_arg);
    float acc = to_f<T>(h[q]);
    for (int j = 0; j < taps; ++j) {
      const int back = taps - 1 - j, p = T0 + s - back;
      if (p < 0) continue;
      const float v = s >= back ? to_f<T>(h[q - (int64_t)back * d]) : to_f<T>(ring[((int64_t)b * taps + p % taps) * d + i]);
      acc += to_f<T>(wgt[(int64_t)i * taps + j]) * v;
    }
    out[q] = from_f<T>(acc);
  }
}
// up to four taps, widths that are multiples of four: four channels and a strip of positions per thread, the window in registers
constexpr int kConvStrip = 16;
template <typename T>
__global__ void __launch_bounds__(128) short_conv_strip_kernel(T* out, const T* h, const T* wgt, const T* ring, int S, int d, int taps, int T0_arg,
                                                               const int* state) {
  const int i = (blockIdx.x * 128 + threadIdx.x) * 4, s0 = blockIdx.y * kConvStrip, b = blockIdx.z;
  if (i >= d) return;
  const int T0 = state_len(state, b, T0_arg);
  float cw[4][4];   // [positions back][channel]
#pragma unroll
  for (int q = 0; q < 4; ++q)
#pragma unroll
    for (int e = 0; e < 4; ++e) cw[q][e] = q < taps ? to_f<T>(wgt[(int64_t)(i + e) * taps + taps - 1 - q]) : 0.0f;
  const T* hb = h + (int64_t)b * S * d + i;
  T* ob = out + (int64_t)b * S * d + i;
  float past[3][4];
#pragma unroll
  for (int q = 1; q < 4; ++q) {
    const int s = s0 - q, p = T0 + s;
    past[q - 1][0] = past[q - 1][1] = past[q - 1][2] = past[q - 1][3] = 0.0f;
    if (q < taps && p >= 0) {
      if (s >= 0) VecIO<T, 4>::load(hb + (int64_t)s * d, past[q - 1]);
      else VecIO<T, 4>::load(ring + ((int64_t)b * taps + p % taps) * d + i, past[q - 1]);
    }
  }
#pragma unroll
  for (int k = 0; k < kConvStrip; ++k) {
    const int s = s0 + k;
    if (s >= S) break;
    float x[4], y[4];
    VecIO<T, 4>::load(hb + (int64_t)s * d, x);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float acc = x[e];
#pragma unroll
      for (int q = 3; q >= 1; --q) acc += cw[q][e] * past[q - 1][e];   // oldest first, as in the other kernels
      y[e] = acc + cw[0][e] * x[e];
      past[2][e] = past[1][e];
      past[1][e] = past[0][e];
      past[0][e] = x[e];
    }
    VecIO<T, 4>::store(ob + (int64_t)s * d, y);
  }
}
template <typename T>
__global__ void __launch_bounds__(256) short_conv_state_kernel(T* ring, const T* h, int S, int d, int taps, int T0_arg, const int* state, const int* lens) {
  const int b = blockIdx.y;
  const int T0 = state_len(state, b, T0_arg);
  const int n = lens ? min(max(lens[b], 1), S) : S;
  const int keep = min(n, taps);
  for (int q = blockIdx.x * blockDim.x + threadIdx.x; q < keep * d; q += gridDim.x * blockDim.x) {
    const int s = n - keep + q / d, i = q % d;
    ring[((int64_t)b * taps + (T0 + s) % taps) * d + i] = h[((int64_t)b * S + s) * d + i];
  }
}

// ---- routing by token id ---------------------------------------------------------------------------------------------------
constexpr int kRouteThreads = 512;

// exclusive prefix sum of s_v[0, n) in place, total returned to every thread; s_tmp: 32 ints
__device__ __forceinline__ int block_exclusive_scan(int* s_v, int n, int* s_tmp) {
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, nw = kRouteThreads / 32;
  int carry = 0;
  for (int base = 0; base < n; base += kRouteThreads) {
    const int i = base + tid;
    const int v = i < n ? s_v[i] : 0;
    int x = v;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int y = __shfl_up_sync(0xffffffffu, x, o);
      if (lane >= o) x += y;
    }
    if (lane == 31) s_tmp[w] = x;
    __syncthreads();
    int off = carry, tot = 0;
    for (int q = 0; q < nw; ++q) {
      if (q < w) off += s_tmp[q];
      tot += s_tmp[q];
    }
    if (i < n) s_v[i] = off + x - v;
    carry += tot;
    __syncthreads();
  }
  return carry;
}

// one CTA per expert layer; dynamic shared memory: 3 * max_experts ints
__global__ void __launch_bounds__(kRouteThreads) table_route_kernel(const RouteLayer* layers, const int* ids, int rows, int V, int block_rows) {
  extern __shared__ int s_int[];
  __shared__ int s_tmp[32];
  pdl_trigger();
  pdl_wait();
  const RouteLayer L = layers[blockIdx.x];
  const int E = L.experts, top = L.top, n = rows * top, tid = threadIdx.x;
  int* cnt = s_int;             // picks per expert
  int* first = s_int + E;       // first sorted row of an expert
  int* blk = s_int + 2 * E;     // first block of an expert
  for (int e = tid; e < E; e += kRouteThreads) cnt[e] = 0;
  __syncthreads();
  auto expert_of = [&](int p) {
    int id = ids[p / top];
    TSB_DEV_CHECK(blocks, id >= 0 && id < V, 0x501, (void)0)   // token id outside the vocabulary (routed as id 0)
    if (id < 0 || id >= V) id = 0;
    int e = L.table[(int64_t)id * top + p % top];
    TSB_DEV_CHECK(blocks, e >= 0 && e < E, 0x502, (void)0)     // the table names an expert that does not exist (checked when it is loaded)
    return min(max(e, 0), E - 1);
  };
  for (int p = tid; p < n; p += kRouteThreads) atomicAdd(&cnt[expert_of(p)], 1);
  __syncthreads();
  for (int e = tid; e < E; e += kRouteThreads) {
    first[e] = cnt[e];
    blk[e] = (cnt[e] + block_rows - 1) / block_rows;
  }
  __syncthreads();
  block_exclusive_scan(first, E, s_tmp);
  const int n_blocks = block_exclusive_scan(blk, E, s_tmp);
  for (int e = tid; e < E; e += kRouteThreads) {
    for (int q = 0; q * block_rows < cnt[e]; ++q) {
      RowBlock rb;
      rb.matrix = e;
      rb.row0 = first[e] + q * block_rows;
      rb.rows = min(block_rows, cnt[e] - q * block_rows);
      rb.pad = 0;
      L.blocks[blk[e] + q] = rb;
    }
  }
  if (tid == 0) *L.n_blocks = n_blocks;
  __syncthreads();
  // the order inside an expert is of no consequence: every row is computed by itself
  for (int p = tid; p < n; p += kRouteThreads) {
    const int e = expert_of(p);
    const int at = atomicAdd(&first[e], 1);
    L.pos[p] = at;
    L.matrix_of[at] = e;
  }
}

// y[r] = epilogue(x[r] W_{matrix_of[r]}) for packed matrices, two columns per thread
template <typename T>
__global__ void __launch_bounds__(128) pick_linear_kernel(const T* x, const T* Wp, const int* matrix_of, int64_t matrix_elems, int K, int N, Epilogue ep) {
  extern __shared__ float s_x[];
  constexpr int NT = sizeof(T) == 2 ? 256 : 128;
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x, KB = (K + 31) / 32;
  for (int i = threadIdx.x; i < K; i += 128) s_x[i] = to_f<T>(x[(int64_t)r * K + i]);
  __syncthreads();
  const int c = (blockIdx.y * 128 + threadIdx.x) * 2;
  if (c >= N) return;
  const T* W = Wp + (int64_t)matrix_of[r] * matrix_elems + (int64_t)(c / NT) * KB * (32 * NT);
  const int cc = c % NT;
  float a0 = 0.0f, a1 = 0.0f;
#pragma unroll 4
  for (int k = 0; k < K; ++k) {
    const T* wp = W + (int64_t)(k >> 5) * (32 * NT) + packed_tile_off<T>(k & 31, cc);   // c is even: its neighbour is the next element
    a0 = fmaf(s_x[k], to_f<T>(wp[0]), a0);
    a1 = fmaf(s_x[k], to_f<T>(wp[1]), a1);
  }
  const T* bias = reinterpret_cast<const T*>(ep.bias);
  const float b0 = bias ? to_f<T>(bias[c]) : 0.0f, b1 = bias && c + 1 < N ? to_f<T>(bias[c + 1]) : 0.0f;
  if (ep.glu) {
    if (c + 1 < N) ep_store<T>(ep, (size_t)r * (N / 2) + (c >> 1), ep_glu(a0 + b0, a1 + b1, ep));
  } else {
    ep_store<T>(ep, (size_t)r * N + c, ep_act(a0 + b0, ep.act));
    if (c + 1 < N) ep_store<T>(ep, (size_t)r * N + c + 1, ep_act(a1 + b1, ep.act));
  }
}

// ---- host side -------------------------------------------------------------------------------------------------------------
int launch_block_norm(int device, int dtype, const BlockNormArgs& a, int out_rows, cudaStream_t s) {
  if (out_rows == 0) return 1;
  TSB_CHECK(a.groups >= 1 && a.d % a.groups == 0, "block_norm: a width of %d is not cut into %d groups", a.d, a.groups);
  if (block_norm_fast_shape(a)) {
    const int nv = a.d <= 2048 ? 1 : 2;
    const dim3 th(a.d / 4 / nv);
#define TSB_BNF(T)                                                                                                                    \
  (a.conv_ring ? (nv == 1 ? block_norm_fast_kernel<T, 1, 4> : block_norm_fast_kernel<T, 2, 4>)                                        \
               : (nv == 1 ? block_norm_fast_kernel<T, 1, 0> : block_norm_fast_kernel<T, 2, 0>))
    if (dtype == TSB200_F32) TSB_CUDA(launch_k(TSB_BNF(float), dim3(out_rows), th, 0, s, a));
    else TSB_CUDA(launch_k(TSB_BNF(__nv_bfloat16), dim3(out_rows), th, 0, s, a));
#undef TSB_BNF
    count_launch(device);
    return check_launch("block_norm_fast");
  }
  const size_t smem = ((size_t)a.d + (a.groups > 8 ? a.groups : 8)) * sizeof(float);
  TSB_CHECK(smem <= 200 * 1024, "block_norm: rows of %d elements are not supported", a.d);
  static bool done[kMaxDevices] = {};
  if (!done[device]) {
    TSB_CUDA(cudaFuncSetAttribute(block_norm_kernel<float, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    TSB_CUDA(cudaFuncSetAttribute(block_norm_kernel<float, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    TSB_CUDA(cudaFuncSetAttribute(block_norm_kernel<__nv_bfloat16, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    TSB_CUDA(cudaFuncSetAttribute(block_norm_kernel<__nv_bfloat16, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    done[device] = true;
  }
  const bool v4 = a.d % 4 == 0;
  if (dtype == TSB200_F32)
    TSB_CUDA(launch_k(v4 ? block_norm_kernel<float, 4> : block_norm_kernel<float, 1>, dim3(out_rows), dim3(kBlockNormThreads), smem, s, a));
  else
    TSB_CUDA(launch_k(v4 ? block_norm_kernel<__nv_bfloat16, 4> : block_norm_kernel<__nv_bfloat16, 1>, dim3(out_rows), dim3(kBlockNormThreads), smem, s, a));
  count_launch(device);
  return check_launch("block_norm");
}

template <typename T, int V>
static cudaError_t sandwich_go(const SandwichNormArgs& a, int out_rows, cudaStream_t s) {
  const int units = (a.d + V - 1) / V;
  int nt = units >= 512 ? 512 : (units + 31) / 32 * 32;
  const int nv = (units + nt - 1) / nt;
  const dim3 g(out_rows), b(nt);
  if (nv <= 1) return launch_k(sandwich_norm_kernel<T, V, 1>, g, b, 0, s, a);
  if (nv <= 2) return launch_k(sandwich_norm_kernel<T, V, 2>, g, b, 0, s, a);
  if (nv <= 4) return launch_k(sandwich_norm_kernel<T, V, 4>, g, b, 0, s, a);
  return launch_k(sandwich_norm_kernel<T, V, 8>, g, b, 0, s, a);
}

int launch_sandwich_norm(int device, int dtype, const SandwichNormArgs& a, int out_rows, cudaStream_t s) {
  if (out_rows == 0) return 1;
  const bool v4 = a.d % 4 == 0;
  TSB_CHECK(a.d > 0 && a.d <= (v4 ? 16384 : 4096), "sandwich_norm: rows of %d elements are not supported", a.d);
  if (dtype == TSB200_F32) TSB_CUDA((v4 ? sandwich_go<float, 4>(a, out_rows, s) : sandwich_go<float, 1>(a, out_rows, s)));
  else TSB_CUDA((v4 ? sandwich_go<__nv_bfloat16, 4>(a, out_rows, s) : sandwich_go<__nv_bfloat16, 1>(a, out_rows, s)));
  count_launch(device);
  return check_launch("sandwich_norm");
}

int launch_short_conv(int device, DeviceState* st, int dtype, void* out, const void* h, const void* w, void* ring, int B, int S, int d, int taps,
                      int T0, const int* state, const int* lens, cudaStream_t s) {
  int64_t g = ((int64_t)B * S * d + 255) / 256;
  if (g > (int64_t)st->sm_count * 32) g = (int64_t)st->sm_count * 32;
  const dim3 g2((unsigned)((taps * d + 255) / 256), B);
  const bool strip = taps <= 4 && d % 4 == 0 && B <= 65535 && (S + kConvStrip - 1) / kConvStrip <= 65535;
  const dim3 gs((d / 4 + 127) / 128, (S + kConvStrip - 1) / kConvStrip, B);
  if (dtype == TSB200_F32) {
    if (strip) short_conv_strip_kernel<float><<<gs, 128, 0, s>>>((float*)out, (const float*)h, (const float*)w, (const float*)ring, S, d, taps, T0, state);
    else short_conv_kernel<float><<<(int)g, 256, 0, s>>>((float*)out, (const float*)h, (const float*)w, (const float*)ring, B, S, d, taps, T0, state);
    short_conv_state_kernel<float><<<g2, 256, 0, s>>>((float*)ring, (const float*)h, S, d, taps, T0, state, lens);
  } else {
    typedef __nv_bfloat16 H;
    if (strip) short_conv_strip_kernel<H><<<gs, 128, 0, s>>>((H*)out, (const H*)h, (const H*)w, (const H*)ring, S, d, taps, T0, state);
    else short_conv_kernel<H><<<(int)g, 256, 0, s>>>((H*)out, (const H*)h, (const H*)w, (const H*)ring, B, S, d, taps, T0, state);
    short_conv_state_kernel<H><<<g2, 256, 0, s>>>((H*)ring, (const H*)h, S, d, taps, T0, state, lens);
  }
  count_launch(device, 2);
  return check_launch("short_conv");
}

int launch_table_route(int device, const RouteLayer* layers_dev, int n_layers, int max_experts, const int* ids, int rows, int V, int block_rows,
                       cudaStream_t s) {
  if (n_layers == 0 || rows == 0) return 1;
  const size_t smem = (size_t)3 * max_experts * sizeof(int);
  TSB_CHECK(smem <= 48 * 1024, "table_route: %d experts are not supported (at most 4096)", max_experts);
  TSB_CUDA(launch_k(table_route_kernel, dim3(n_layers), dim3(kRouteThreads), smem, s, layers_dev, ids, rows, V, block_rows));
  count_launch(device);
  return check_launch("table_route");
}

int launch_pick_linear(int device, int dtype, const void* x, const void* Wp, const int* matrix_of, int64_t matrix_bytes, int rows, int K, int N,
                       const Epilogue& ep, cudaStream_t s) {
  if (rows == 0) return 1;
  const size_t smem = (size_t)K * sizeof(float);
  TSB_CHECK(smem <= 48 * 1024, "pick_linear: rows of %d inputs are not supported", K);
  const dim3 grid(rows, (N + 255) / 256);
  if (dtype == TSB200_F32)
    TSB_CUDA(launch_k(pick_linear_kernel<float>, grid, dim3(128), smem, s, (const float*)x, (const float*)Wp, matrix_of, matrix_bytes / 4, K, N, ep));
  else
    TSB_CUDA(launch_k(pick_linear_kernel<__nv_bfloat16>, grid, dim3(128), smem, s, (const __nv_bfloat16*)x, (const __nv_bfloat16*)Wp, matrix_of,
                      matrix_bytes / 2, K, N, ep));
  count_launch(device);
  return check_launch("pick_linear");
}

}  // namespace tsb
