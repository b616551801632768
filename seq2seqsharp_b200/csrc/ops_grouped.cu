// Grouped-query attention with everything that layered designs put around the softmax, each part optional and with its constants as
// parameters:
//   per-head RMS norm of queries and keys; a sliding window with kept first tokens; a learned bias by distance; a sink (a logit per head
//   that joins the denominator without a key or a value); a gate per head on the output.
//
//   score(i, j) = scale (q_i . k_j) + bias[h][min(i - j, n_bias - 1)],   j <= i and (i - j < window or j < keep_first)
//   out_i = sigmoid(g_h) sum_j e^score v_j / (sum_j e^score + e^sink_h)
//
// Cache: keys [sequences][G][Tmax][dk] after their norm, values [sequences][G][Tmax][dv], rows rounded up to 8 elements (the rest stays
// zero).  A layer may read another layer's cache.
//
// The visible keys of a query are two pieces, the kept first tokens and the window; kernels walk one list that joins them
// (KeyList), so nothing between the pieces is touched.
//   head_prep_kernel          norms queries into a scratch, appends the normed keys and the values (prompts, and every CUDA-core step)
//   grouped_prefill_kernel    bf16 prompts: 64 (query, head) rows of one key/value head per CTA, keys and values staged once, mma.sync
//   grouped_decode_kernel     bf16, one new position per sequence: norm and append of the projected row, attention over a split of
//                             the key list and, in the CTA that finishes last, the merge with sink and gate - one launch
//   grouped_simple_kernel     any type and size, CUDA cores
// Scores, bias, softmax and sums are fp32 in every kernel; the softmax weights are rounded to bf16 as operands of the tensor cores.
#include <algorithm>

#include "kernels.cuh"
#include "warp_tiles.cuh"

namespace tsb {

TSB_CHECKED_WORD(grouped)
#ifndef TSB200_CHECKED
int chk_take_grouped() { return 0; }
#endif

// The keys that queries at positions first .. last see (all of them together), in order: [0, kept) and [lo, last].
struct KeyList {
  int kept, lo, n;
  __device__ __forceinline__ KeyList(const GroupedShape& a, int first, int last) {
    lo = a.window > 0 ? max(0, first - a.window + 1) : 0;
    kept = min(a.keep_first, lo);
    n = kept + last - lo + 1;
  }
  __device__ __forceinline__ int at(int u) const { return u < kept ? u : u - kept + lo; }
};
__device__ __forceinline__ bool key_visible(const GroupedShape& a, int i, int j) {
  return j <= i && (a.window <= 0 || i - j < a.window || j < a.keep_first);
}
__device__ __forceinline__ float head_gate(float g) { return 1.0f / (1.0f + expf(-g)); }

// ---- norm of queries and keys, cache append: one warp per (row, head) -------------------------------------------------------------
template <typename T, int V>
struct HeadVec {
  static __device__ __forceinline__ void load(const T* p, float* f) {
#pragma unroll
    for (int e = 0; e < V; ++e) f[e] = to_f<T>(p[e]);
  }
  static __device__ __forceinline__ void store(T* p, const float* f) {
#pragma unroll
    for (int e = 0; e < V; ++e) p[e] = from_f<T>(f[e]);
  }
};
template <>
struct HeadVec<bf16, 4> {
  static __device__ __forceinline__ void load(const bf16* p, float* f) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = Pair16<bf16>::get(t.x), b = Pair16<bf16>::get(t.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  }
  static __device__ __forceinline__ void store(bf16* p, const float* f) {
    *reinterpret_cast<uint2*>(p) = make_uint2(Pair16<bf16>::put(f[0], f[1]), Pair16<bf16>::put(f[2], f[3]));
  }
};
template <>
struct HeadVec<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float* f) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    f[0] = t.x; f[1] = t.y; f[2] = t.z; f[3] = t.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};

template <typename T, int V>
__global__ void __launch_bounds__(256) head_prep_kernel(GroupedArgs a) {
  pdl_trigger();
  pdl_wait();
  const GroupedShape& sh = a.shape;
  const int lane = threadIdx.x & 31;
  const int units = sh.H + (a.k_col >= 0 ? 2 * sh.G : 0);
  const unsigned n_all = (unsigned)(a.B * a.S) * (unsigned)units;
  for (unsigned w = blockIdx.x * 8 + (threadIdx.x >> 5); w < n_all; w += gridDim.x * 8) {
    const unsigned r = w / (unsigned)units;
    const int u = (int)(w - r * (unsigned)units);
    const int64_t row = r;
    const int b = (int)(r / (unsigned)a.S), pos = state_len(a.state, b, a.T0) + (int)(r % (unsigned)a.S);
    TSB_DEV_CHECK(grouped, pos >= 0 && pos < a.Tmax, 0x601, (void)0)   // append position outside the cache (row skipped)
    const T* src = reinterpret_cast<const T*>(a.qkv) + row * a.q_stride;
    const T* wt = nullptr;
    T* dst;
    int n = sh.dim;
    if (u < sh.H) {
      src += (int64_t)u * sh.dim;
      dst = reinterpret_cast<T*>(a.qn) + (row * sh.H + u) * sh.dk;
      wt = reinterpret_cast<const T*>(a.q_norm);
    } else {
      if (pos >= a.Tmax) continue;
      const int g = (u - sh.H) % sh.G;
      if (u < sh.H + sh.G) {
        src += a.k_col + (int64_t)g * sh.dim;
        dst = reinterpret_cast<T*>(a.cK) + (((int64_t)b * sh.G + g) * a.Tmax + pos) * sh.dk;
        wt = reinterpret_cast<const T*>(a.k_norm);
      } else {
        n = sh.vdim;
        src += a.v_col + (int64_t)g * sh.vdim;
        dst = reinterpret_cast<T*>(a.cV) + (((int64_t)b * sh.G + g) * a.Tmax + pos) * sh.dv;
      }
    }
    if (n <= 32 * V) {   // the row in registers
      float v[V], g[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {
        v[e] = 0.0f;
        g[e] = 1.0f;
      }
      const int i = lane * V;
      if (i < n) {
        HeadVec<T, V>::load(src + i, v);
        if (wt) HeadVec<T, V>::load(wt + i, g);
      }
      if (wt) {
        float s = 0.0f;
#pragma unroll
        for (int e = 0; e < V; ++e) s += v[e] * v[e];
        const float inv = 1.0f / sqrtf(warp_sum(s) / (float)n + sh.eps);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = v[e] * inv * g[e];
      }
      if (i < n) HeadVec<T, V>::store(dst + i, v);
      if (u < sh.H)
        for (int e = n + lane; e < sh.dk; e += 32) dst[e] = from_f<T>(0.0f);
      continue;
    }
    float inv = 1.0f;
    if (wt) {
      float s = 0.0f;
      for (int i = lane * V; i < n; i += 32 * V) {
        float v[V];
        HeadVec<T, V>::load(src + i, v);
#pragma unroll
        for (int e = 0; e < V; ++e) s += v[e] * v[e];
      }
      inv = 1.0f / sqrtf(warp_sum(s) / (float)n + sh.eps);
    }
    for (int i = lane * V; i < n; i += 32 * V) {
      float v[V];
      HeadVec<T, V>::load(src + i, v);
      if (wt) {
        float g[V];
        HeadVec<T, V>::load(wt + i, g);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = v[e] * inv * g[e];
      }
      HeadVec<T, V>::store(dst + i, v);
    }
    if (u < sh.H)
      for (int i = n + lane; i < sh.dk; i += 32) dst[i] = from_f<T>(0.0f);
  }
}

// ---- any type and size: one CTA per (row, head) ------------------------------------------------------------------------------------
constexpr int kGsimThreads = 128;
template <typename T>
__global__ void __launch_bounds__(kGsimThreads) grouped_simple_kernel(GroupedArgs a) {
  extern __shared__ float s_f[];   // query [dk], result [vdim], weights [128], 32 for sums
  const GroupedShape& sh = a.shape;
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
  const int64_t row = blockIdx.y;
  const int b = (int)(row / a.S), p = state_len(a.state, b, a.T0) + (int)(row % a.S);
  TSB_DEV_CHECK(grouped, p >= 0 && p < a.Tmax, 0x602, return)   // query position outside the cache
  if (p >= a.Tmax) return;
  float *s_q = s_f, *s_acc = s_q + sh.dk, *s_p = s_acc + sh.vdim, *s_red = s_p + kGsimThreads;
  const T* q = reinterpret_cast<const T*>(a.qn) + (row * sh.H + h) * sh.dk;
  for (int i = tid; i < sh.dk; i += kGsimThreads) s_q[i] = to_f<T>(q[i]);
  for (int i = tid; i < sh.vdim; i += kGsimThreads) s_acc[i] = 0.0f;
  const int g = h / (sh.H / sh.G);
  const T* K = reinterpret_cast<const T*>(a.cK) + ((int64_t)b * sh.G + g) * a.Tmax * sh.dk;
  const T* V = reinterpret_cast<const T*>(a.cV) + ((int64_t)b * sh.G + g) * a.Tmax * sh.dv;
  const float* bias = sh.n_bias > 0 ? a.bias + (int64_t)h * sh.n_bias : nullptr;
  const KeyList keys(sh, p, p);
  // the sink is the first entry of the running softmax
  float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.0f : 0.0f;
  __syncthreads();
  for (int u0 = 0; u0 < keys.n; u0 += kGsimThreads) {
    const int cnt = min(kGsimThreads, keys.n - u0);
    for (int t = w; t < cnt; t += kGsimThreads / 32) {
      const int j = keys.at(u0 + t);
      const T* k = K + (int64_t)j * sh.dk;
      float d = 0.0f;
      for (int i = lane; i < sh.dim; i += 32) d = fmaf(s_q[i], to_f<T>(k[i]), d);
      d = warp_sum(d) * sh.scale;
      if (bias) d += bias[min(p - j, sh.n_bias - 1)];
      if (lane == 0) s_p[t] = d;
    }
    __syncthreads();
    const float z = tid < cnt ? s_p[tid] : -INFINITY;
    const float mn = fmaxf(m, block_max(z, s_red));
    const float e = tid < cnt ? expf(z - mn) : 0.0f, corr = expf(m - mn);
    l = l * corr + block_sum(e, s_red);
    m = mn;
    s_p[tid] = e;
    __syncthreads();
    for (int c = tid; c < sh.vdim; c += kGsimThreads) {
      float acc = s_acc[c] * corr;
      for (int t = 0; t < cnt; ++t) acc = fmaf(s_p[t], to_f<T>(V[(int64_t)keys.at(u0 + t) * sh.dv + c]), acc);
      s_acc[c] = acc;
    }
    __syncthreads();
  }
  float f = 1.0f / l;
  if (a.g_col >= 0) f *= head_gate(to_f<T>(reinterpret_cast<const T*>(a.qkv)[row * a.q_stride + a.g_col + h]));
  T* out = reinterpret_cast<T*>(a.out) + (row * sh.H + h) * sh.vdim;
  for (int c = tid; c < sh.vdim; c += kGsimThreads) out[c] = from_f<T>(s_acc[c] * f);
}

// ---- bf16 tensor-core kernels -------------------------------------------------------------------------------------------------------
// Staged rows are D elements (dim and vdim rounded up to one of a few sizes, zero beyond) plus 16 bytes, so that the eight rows of an
// ldmatrix fall into different banks.
constexpr int kGaThreads = 128, kGaKeys = 64, kGaStages = 2;   // two stages: more CTAs per SM hide more than a third stage would

template <int D> struct GaTile {
  static constexpr int pitch = D * 2 + 16;
  static constexpr uint32_t plane = (uint32_t)kGaKeys * pitch;   // keys, or values, of a stage
  static constexpr uint32_t stage = 2 * plane;
};
// The 16-byte units of a stage's rows that a thread copies, walked without divisions.
struct UnitWalk {
  int r0, c0, dr, dc, cols;
  __device__ __forceinline__ explicit UnitWalk(int n) : cols(n) {
    r0 = threadIdx.x / n;
    c0 = threadIdx.x % n;
    dr = kGaThreads / n;
    dc = kGaThreads % n;
  }
  template <typename F>
  __device__ __forceinline__ void each(F f) const {
    for (int r = r0, c = c0; r < kGaKeys;) {
      f(r, c);
      r += dr;
      c += dc;
      if (c >= cols) {
        c -= cols;
        ++r;
      }
    }
  }
};
// zeros into the columns that no copy writes
template <int D>
__device__ __forceinline__ void ga_zero_pads(unsigned char* smem, int stages, int dk, int dv) {
  const int kc = dk / 8, vc = dv / 8, per = (D / 8 - kc) + (D / 8 - vc);
  if (per == 0) return;
  for (int v = threadIdx.x; v < stages * kGaKeys * per; v += kGaThreads) {
    const int s = v / (kGaKeys * per), r = v / per % kGaKeys, c = v % per;
    const bool val = c >= D / 8 - kc;
    unsigned char* p = smem + s * GaTile<D>::stage + (val ? GaTile<D>::plane : 0) + r * GaTile<D>::pitch + (val ? vc + c - (D / 8 - kc) : kc + c) * 16;
    *reinterpret_cast<uint4*>(p) = make_uint4(0u, 0u, 0u, 0u);
  }
}

// grid (tiles of qt query positions, key/value heads x chunks of hp query heads, sequences)
template <int D>
__global__ void __launch_bounds__(kGaThreads, D <= 64 ? 4 : D <= 128 ? 3 : 1) grouped_prefill_kernel(GroupedArgs a, int hp, int qt, int bias_in_smem) {
  constexpr int PITCH = GaTile<D>::pitch, KS = D / 16, NBO = D / 8;
  extern __shared__ __align__(128) unsigned char smem[];
  const GroupedShape& sh = a.shape;
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, g8 = lane >> 2, t4 = lane & 3;
  const int group = sh.H / sh.G, chunks = gridDim.y / sh.G;
  const int kvh = blockIdx.y / chunks, gh0 = (blockIdx.y % chunks) * hp;
  const int b = blockIdx.z, q0 = blockIdx.x * qt;
  const int T0 = state_len(a.state, b, a.T0);
  const int n_q = min(qt, a.S - q0);
  const int p_first = T0 + q0, p_last = min(T0 + q0 + n_q, a.Tmax) - 1;
  const KeyList keys(sh, p_first, p_last);
  const int n_tiles = (keys.n + kGaKeys - 1) / kGaKeys;
  const bf16* Kb = reinterpret_cast<const bf16*>(a.cK) + ((int64_t)b * sh.G + kvh) * a.Tmax * sh.dk;
  const bf16* Vb = reinterpret_cast<const bf16*>(a.cV) + ((int64_t)b * sh.G + kvh) * a.Tmax * sh.dv;
  const uint32_t s0 = la_smem(smem);
  const UnitWalk walk_k(sh.dk / 8), walk_v(sh.dv / 8);

  auto issue = [&](int tile) {
    if (tile < n_tiles) {
      const uint32_t st = s0 + (uint32_t)(tile % kGaStages) * GaTile<D>::stage;
      walk_k.each([&](int r, int c) {
        const int u = tile * kGaKeys + r;
        la_cp16(st + r * PITCH + c * 16, Kb + (int64_t)keys.at(min(u, keys.n - 1)) * sh.dk + c * 8, u < keys.n);
      });
      walk_v.each([&](int r, int c) {
        const int u = tile * kGaKeys + r;
        la_cp16(st + GaTile<D>::plane + r * PITCH + c * 16, Vb + (int64_t)keys.at(min(u, keys.n - 1)) * sh.dv + c * 8, u < keys.n);
      });
    }
    la_commit();
  };
  for (int i = 0; i < kGaStages - 1; ++i) issue(i);
  ga_zero_pads<D>(smem, kGaStages, sh.dk, sh.dv);

  // this lane's two rows, (query, head) pairs; scores, maxima and bias in powers of two
  int pos[2], head[2];
  bool live[2];
  const float* bias[2];
  float far_bias[2];   // of every distance from n_bias - 1 on
  const float bias_unit = bias_in_smem ? 1.0f : kLog2e, scale = sh.scale * kLog2e;
  float* s_bias = reinterpret_cast<float*>(smem + kGaStages * GaTile<D>::stage);
  uint32_t qa[KS][4];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int rr = w * 16 + g8 + r * 8, qi = rr / hp, gh = gh0 + rr % hp;
    live[r] = qi < n_q && gh < group;
    pos[r] = T0 + q0 + (live[r] ? qi : 0);
    head[r] = kvh * group + (live[r] ? gh : gh0);
    bias[r] = bias_in_smem ? s_bias + (live[r] ? rr % hp : 0) * sh.n_bias : a.bias + (int64_t)head[r] * sh.n_bias;
    far_bias[r] = sh.n_bias > 0 ? a.bias[(int64_t)head[r] * sh.n_bias + sh.n_bias - 1] * kLog2e : 0.0f;
    const bf16* qp = reinterpret_cast<const bf16*>(a.qn) + (((int64_t)b * a.S + pos[r] - T0) * sh.H + head[r]) * sh.dk + 2 * t4;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      qa[ks][r] = live[r] && ks * 16 < sh.dk ? *reinterpret_cast<const uint32_t*>(qp + ks * 16) : 0u;
      qa[ks][r + 2] = live[r] && ks * 16 + 8 < sh.dk ? *reinterpret_cast<const uint32_t*>(qp + ks * 16 + 8) : 0u;
    }
  }
  if (bias_in_smem)
    for (int i = threadIdx.x; i < min(hp, group - gh0) * sh.n_bias; i += kGaThreads) s_bias[i] = a.bias[(int64_t)(kvh * group + gh0) * sh.n_bias + i] * kLog2e;
  // this warp's range of query positions
  const int wq0 = (w * 16) / hp, wq1 = min((w * 16 + 15) / hp, n_q - 1);
  const int wp0 = T0 + q0 + wq0, wp1 = T0 + q0 + wq1;
  float m[2], l[2], o[NBO][4];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    m[r] = a.sink ? a.sink[head[r]] * kLog2e : -INFINITY;
    l[r] = a.sink && t4 == 0 ? 1.0f : 0.0f;   // the quad's parts are added at the end
  }
#pragma unroll
  for (int nb = 0; nb < NBO; ++nb)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[nb][e] = 0.0f;

  for (int tile = 0; tile < n_tiles; ++tile) {
    issue(tile + kGaStages - 1);
    la_wait<kGaStages - 1>();
    __syncthreads();
    const uint32_t kb = s0 + (uint32_t)(tile % kGaStages) * GaTile<D>::stage, vb = kb + GaTile<D>::plane;
#pragma unroll 1
    for (int sl = 0; sl < kGaKeys / 32; ++sl) {
      const int u0 = tile * kGaKeys + sl * 32;
      if (u0 >= keys.n || wq0 >= n_q) break;
      const int ja = keys.at(u0), jb = keys.at(min(u0 + 31, keys.n - 1));
      if (ja > wp1) break;   // later keys are later positions: nothing more for this warp
      if (sh.window > 0 && ja >= sh.keep_first && jb <= wp0 - sh.window) continue;
      const int tw = sl * 32;
      float sc[4][4];
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[nb][e] = 0.0f;
      const uint32_t ka = kb + (tw + (lane & 7)) * PITCH + (lane >> 3) * 16;
#pragma unroll
      for (int kp = 0; kp < KS / 2; ++kp) {   // four independent sums side by side
        uint32_t kf[4][4];
#pragma unroll
        for (int nb = 0; nb < 4; ++nb) la_ldsm_x4(ka + nb * 8 * PITCH + kp * 64, kf[nb][0], kf[nb][1], kf[nb][2], kf[nb][3]);
#pragma unroll
        for (int nb = 0; nb < 4; ++nb) la_mma(sc[nb], qa[2 * kp][0], qa[2 * kp][1], qa[2 * kp][2], qa[2 * kp][3], kf[nb][0], kf[nb][1]);
#pragma unroll
        for (int nb = 0; nb < 4; ++nb) la_mma(sc[nb], qa[2 * kp + 1][0], qa[2 * kp + 1][1], qa[2 * kp + 1][2], qa[2 * kp + 1][3], kf[nb][2], kf[nb][3]);
      }
      // row r: elements 2r, 2r + 1 of every block; keys nb * 8 + 2 * t4 + e
      const bool all_seen = u0 + 31 < keys.n && jb <= wp0 && (sh.window <= 0 || wp1 - ja < sh.window || jb < sh.keep_first);
      if (all_seen && wp0 - jb >= sh.n_bias - 1) {   // (most slices) nothing to mask, one bias for all distances
#pragma unroll
        for (int nb = 0; nb < 4; ++nb)
#pragma unroll
          for (int e = 0; e < 4; ++e) sc[nb][e] = fmaf(sc[nb][e], scale, far_bias[e >> 1]);
      } else {
#pragma unroll
        for (int nb = 0; nb < 4; ++nb)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int u = u0 + nb * 8 + 2 * t4 + e, j = keys.at(u);
#pragma unroll
            for (int r = 0; r < 2; ++r) {
              const bool vis = live[r] && u < keys.n && key_visible(sh, pos[r], j);
              float z = sc[nb][2 * r + e] * scale;
              if (sh.n_bias > 0) z += bias[r][min(max(pos[r] - j, 0), sh.n_bias - 1)] * bias_unit;
              sc[nb][2 * r + e] = vis ? z : -INFINITY;
            }
          }
      }
      float corr[2];
      bool moved = false;
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float mx = -INFINITY;
#pragma unroll
        for (int nb = 0; nb < 4; ++nb) mx = fmaxf(mx, fmaxf(sc[nb][2 * r], sc[nb][2 * r + 1]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float mn = fmaxf(m[r], mx), base = mn == -INFINITY ? 0.0f : mn;   // a row that has seen nothing yet: all weights 0
        corr[r] = exp2_fast(m[r] - base);
        moved = moved || mn != m[r];
        float s = 0.0f;
#pragma unroll
        for (int nb = 0; nb < 4; ++nb)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            sc[nb][2 * r + e] = exp2_fast(sc[nb][2 * r + e] - base);
            s += sc[nb][2 * r + e];
          }
        l[r] = l[r] * corr[r] + s;
        m[r] = mn;
      }
      if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
        for (int nb = 0; nb < NBO; ++nb)
#pragma unroll
          for (int e = 0; e < 4; ++e) o[nb][e] *= corr[e >> 1];
      }
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const uint32_t pa0 = Pair16<bf16>::put(sc[2 * hh][0], sc[2 * hh][1]), pa1 = Pair16<bf16>::put(sc[2 * hh][2], sc[2 * hh][3]);
        const uint32_t pa2 = Pair16<bf16>::put(sc[2 * hh + 1][0], sc[2 * hh + 1][1]), pa3 = Pair16<bf16>::put(sc[2 * hh + 1][2], sc[2 * hh + 1][3]);
        const uint32_t va = vb + (tw + hh * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PITCH + (lane >> 4) * 16;
#pragma unroll
        for (int np = 0; np < NBO / 2; ++np) {
          uint32_t b0, b1, b2, b3;
          la_ldsm_x4_trans(va + np * 32, b0, b1, b2, b3);
          la_mma(o[2 * np], pa0, pa1, pa2, pa3, b0, b1);
          la_mma(o[2 * np + 1], pa0, pa1, pa2, pa3, b2, b3);
        }
      }
    }
    __syncthreads();   // the stage is overwritten by the copy issued in the next iteration
  }
  la_wait<0>();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    if (!live[r]) continue;
    const int64_t row = (int64_t)b * a.S + pos[r] - T0;
    float f = l[r] > 0.0f ? 1.0f / l[r] : 0.0f;
    if (a.g_col >= 0) f *= head_gate(to_f<bf16>(reinterpret_cast<const bf16*>(a.qkv)[row * a.q_stride + a.g_col + head[r]]));
    bf16* op = reinterpret_cast<bf16*>(a.out) + (row * sh.H + head[r]) * sh.vdim + 2 * t4;
#pragma unroll
    for (int nb = 0; nb < NBO; ++nb)
      if (nb * 8 + 2 * t4 < sh.vdim) *reinterpret_cast<uint32_t*>(op + nb * 8) = Pair16<bf16>::put(o[nb][2 * r] * f, o[nb][2 * r + 1] * f);
  }
}

// One new position per sequence.  grid (splits, key/value heads x chunks of hp query heads, sequences); hp <= 8 * RH heads are rows of
// the 16-row products.  Every warp owns 16 keys of a stage and a softmax state of its own; the four states meet in shared memory, the
// splits in `part`, where the CTA that finishes last merges them.
template <int D, int RH>
__global__ void __launch_bounds__(kGaThreads) grouped_decode_kernel(GroupedArgs a, int hp) {
  constexpr int PITCH = GaTile<D>::pitch, KS = D / 16, NBO = D / 8, ROWS = 8 * RH, REC = D + 4, NS = kGaStages;
  extern __shared__ __align__(128) unsigned char smem[];   // stages, queries [ROWS] rows, the new key and value row
  __shared__ int s_last;
  const GroupedShape& sh = a.shape;
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
  const int splits = gridDim.x, split = blockIdx.x;
  const int group = sh.H / sh.G, chunks = gridDim.y / sh.G;
  const int kvh = blockIdx.y / chunks, chunk = blockIdx.y % chunks, gh0 = chunk * hp, b = blockIdx.z;
  const int nh = min(hp, group - gh0), h0 = kvh * group + gh0;   // query heads of this CTA
  const int p = min(state_len(a.state, b, a.T0), a.Tmax - 1);
  TSB_DEV_CHECK(grouped, state_len(a.state, b, a.T0) < a.Tmax, 0x603, (void)0)   // the cache is full (the last row is overwritten)
  const KeyList keys(sh, p, p);
  const int per_split = (keys.n + splits - 1) / splits;
  const int u_beg = min(split * per_split, keys.n), u_end = min(keys.n, u_beg + per_split);
  const bool fresh = a.k_col >= 0 && u_beg < keys.n && u_end == keys.n;   // the new position's row is in this split
  const int n_tiles = (u_end - u_beg + kGaKeys - 1) / kGaKeys;
  bf16* Kb = reinterpret_cast<bf16*>(a.cK) + ((int64_t)b * sh.G + kvh) * a.Tmax * sh.dk;
  bf16* Vb = reinterpret_cast<bf16*>(a.cV) + ((int64_t)b * sh.G + kvh) * a.Tmax * sh.dv;
  const uint32_t s0 = la_smem(smem);
  const int kc = sh.dk / 8, vc = sh.dv / 8;
  const UnitWalk walk_k(kc), walk_v(vc);

  auto issue = [&](int tile) {
    if (tile < n_tiles) {
      const uint32_t st = s0 + (uint32_t)(tile % NS) * GaTile<D>::stage;
      walk_k.each([&](int r, int c) {
        const int u = u_beg + tile * kGaKeys + r, j = keys.at(min(u, u_end - 1));
        la_cp16(st + r * PITCH + c * 16, Kb + (int64_t)j * sh.dk + c * 8, u < u_end && !(fresh && j == p));
      });
      walk_v.each([&](int r, int c) {
        const int u = u_beg + tile * kGaKeys + r, j = keys.at(min(u, u_end - 1));
        la_cp16(st + GaTile<D>::plane + r * PITCH + c * 16, Vb + (int64_t)j * sh.dv + c * 8, u < u_end && !(fresh && j == p));
      });
    }
    la_commit();
  };
  for (int i = 0; i < NS - 1; ++i) issue(i);
  ga_zero_pads<D>(smem, NS, sh.dk, sh.dv);

  // while the first rows travel: queries normed into shared memory, the new key and value row into shared memory and the cache
  unsigned char* s_q = smem + NS * GaTile<D>::stage;
  bf16* s_new = reinterpret_cast<bf16*>(s_q + ROWS * PITCH);   // [2][D]
  const bf16* row = reinterpret_cast<const bf16*>(a.qkv) + (int64_t)b * a.q_stride;
  for (int i = tid; i < (ROWS - nh) * (PITCH / 16); i += kGaThreads)   // rows without a head
    reinterpret_cast<uint4*>(s_q + (nh + i / (PITCH / 16)) * PITCH)[i % (PITCH / 16)] = make_uint4(0u, 0u, 0u, 0u);
  const int n_items = nh + (fresh ? 2 : 0);   // query heads, the key row, the value row
  for (int i0 = w; i0 < n_items; i0 += 2 * (kGaThreads / 32)) {
    float v[2][D / 32], g[2][D / 32];
#pragma unroll
    for (int q = 0; q < 2; ++q) {   // two rows requested at a time
      const int it = i0 + q * (kGaThreads / 32);
      const bool is_v = it == nh + 1, is_k = it == nh;
      const int n = it >= n_items ? 0 : (is_v ? sh.vdim : sh.dim);
      const bf16* src = row + (is_v ? a.v_col + kvh * sh.vdim : (is_k ? a.k_col + kvh * sh.dim : (h0 + min(it, nh - 1)) * sh.dim));
      const bf16* wt = reinterpret_cast<const bf16*>(is_v ? nullptr : (is_k ? a.k_norm : a.q_norm));
#pragma unroll
      for (int i = 0; i < D / 32; ++i) {
        const int e = lane + i * 32;
        v[q][i] = e < n ? to_f<bf16>(src[e]) : 0.0f;
        g[q][i] = wt && e < n ? to_f<bf16>(wt[e]) : 1.0f;
      }
    }
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const int it = i0 + q * (kGaThreads / 32);
      if (it >= n_items) break;
      const bool is_v = it == nh + 1, is_k = it == nh;
      const int n = is_v ? sh.vdim : sh.dim, n_pad = is_v ? sh.dv : (is_k ? sh.dk : D);
      float s = 0.0f;
#pragma unroll
      for (int i = 0; i < D / 32; ++i) s += v[q][i] * v[q][i];
      const float inv = !is_v && (is_k ? a.k_norm : a.q_norm) ? 1.0f / sqrtf(warp_sum(s) / (float)n + sh.eps) : 1.0f;
      bf16* dst = is_v ? s_new + D : (is_k ? s_new : reinterpret_cast<bf16*>(s_q + it * PITCH));
      bf16* cache = chunk != 0 || it < nh ? nullptr : (is_k ? Kb + (int64_t)p * sh.dk : Vb + (int64_t)p * sh.dv);
#pragma unroll
      for (int i = 0; i < D / 32; ++i) {
        const int e = lane + i * 32;
        if (e >= n_pad) continue;
        const bf16 t = from_f<bf16>(v[q][i] * inv * g[q][i]);
        dst[e] = t;
        if (cache && e < n) cache[e] = t;
      }
    }
  }
  __syncthreads();
  uint32_t qa[KS][4];
  {
    const unsigned char* qp = s_q + g8 * PITCH + 4 * t4;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      qa[ks][0] = *reinterpret_cast<const uint32_t*>(qp + ks * 32);
      qa[ks][2] = *reinterpret_cast<const uint32_t*>(qp + ks * 32 + 16);
      qa[ks][1] = RH == 2 ? *reinterpret_cast<const uint32_t*>(qp + (RH - 1) * 8 * PITCH + ks * 32) : 0u;
      qa[ks][3] = RH == 2 ? *reinterpret_cast<const uint32_t*>(qp + (RH - 1) * 8 * PITCH + ks * 32 + 16) : 0u;
    }
  }
  const float* bias[RH];
  float far_bias[RH];   // of every distance from n_bias - 1 on
#pragma unroll
  for (int r = 0; r < RH; ++r) {
    bias[r] = a.bias + (int64_t)(h0 + min(g8 + 8 * r, nh - 1)) * sh.n_bias;
    far_bias[r] = sh.n_bias > 0 ? bias[r][sh.n_bias - 1] : 0.0f;
  }
  float m[RH], l[RH], o[NBO][2 * RH];
#pragma unroll
  for (int r = 0; r < RH; ++r) {
    m[r] = -INFINITY;
    l[r] = 0.0f;
  }
#pragma unroll
  for (int nb = 0; nb < NBO; ++nb)
#pragma unroll
    for (int e = 0; e < 2 * RH; ++e) o[nb][e] = 0.0f;

  for (int tile = 0; tile < n_tiles; ++tile) {
    issue(tile + NS - 1);
    la_wait<NS - 1>();
    __syncthreads();
    const uint32_t kb = s0 + (uint32_t)(tile % NS) * GaTile<D>::stage, vb = kb + GaTile<D>::plane;
    if (fresh && tile == n_tiles - 1) {   // the new row takes its place
      unsigned char* st = smem + (tile % NS) * GaTile<D>::stage + ((u_end - 1 - u_beg) % kGaKeys) * PITCH;
      if (tid < kc) reinterpret_cast<uint4*>(st)[tid] = reinterpret_cast<const uint4*>(s_new)[tid];
      else if (tid >= 64 && tid < 64 + vc) reinterpret_cast<uint4*>(st + GaTile<D>::plane)[tid - 64] = reinterpret_cast<const uint4*>(s_new + D)[tid - 64];
      __syncthreads();
    }
    const int tw = w * 16, u0 = u_beg + tile * kGaKeys + tw;
    if (u0 < u_end) {
      float bv[RH][2][2];
#pragma unroll
      for (int r = 0; r < RH; ++r) bv[r][0][0] = bv[r][0][1] = bv[r][1][0] = bv[r][1][1] = far_bias[r];
      if (p - keys.at(min(u0 + 15, u_end - 1)) < sh.n_bias - 1) {
#pragma unroll
        for (int nb = 0; nb < 2; ++nb)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int n = min(p - keys.at(min(u0 + nb * 8 + 2 * t4 + e, u_end - 1)), sh.n_bias - 1);
#pragma unroll
            for (int r = 0; r < RH; ++r) bv[r][nb][e] = bias[r][n];
          }
      }
      float sc[2][4], sd[2][4];   // even and odd steps: four independent sums
#pragma unroll
      for (int nb = 0; nb < 2; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[nb][e] = sd[nb][e] = 0.0f;
      const uint32_t ka = kb + (tw + (lane & 7)) * PITCH + (lane >> 3) * 16;
#pragma unroll
      for (int kp = 0; kp < KS / 2; ++kp) {
        uint32_t kf[2][4];
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) la_ldsm_x4(ka + nb * 8 * PITCH + kp * 64, kf[nb][0], kf[nb][1], kf[nb][2], kf[nb][3]);
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) {
          la_mma(sc[nb], qa[2 * kp][0], qa[2 * kp][1], qa[2 * kp][2], qa[2 * kp][3], kf[nb][0], kf[nb][1]);
          la_mma(sd[nb], qa[2 * kp + 1][0], qa[2 * kp + 1][1], qa[2 * kp + 1][2], qa[2 * kp + 1][3], kf[nb][2], kf[nb][3]);
        }
      }
#pragma unroll
      for (int nb = 0; nb < 2; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[nb][e] += sd[nb][e];
      float corr[RH];
#pragma unroll
      for (int r = 0; r < RH; ++r) {
        float mx = -INFINITY;
#pragma unroll
        for (int nb = 0; nb < 2; ++nb)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            float z = fmaf(sc[nb][2 * r + e], sh.scale, bv[r][nb][e]);
            z = u0 + nb * 8 + 2 * t4 + e < u_end ? z : -INFINITY;
            sc[nb][2 * r + e] = z;
            mx = fmaxf(mx, z);
          }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float mn = fmaxf(m[r], mx);   // finite: the slice has at least one valid key
        corr[r] = __expf(m[r] - mn);
        float s = 0.0f;
#pragma unroll
        for (int nb = 0; nb < 2; ++nb)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            sc[nb][2 * r + e] = __expf(sc[nb][2 * r + e] - mn);
            s += sc[nb][2 * r + e];
          }
        l[r] = l[r] * corr[r] + s;
        m[r] = mn;
      }
      const uint32_t pa0 = Pair16<bf16>::put(sc[0][0], sc[0][1]), pa2 = Pair16<bf16>::put(sc[1][0], sc[1][1]);
      const uint32_t pa1 = RH == 2 ? Pair16<bf16>::put(sc[0][2], sc[0][3]) : 0u, pa3 = RH == 2 ? Pair16<bf16>::put(sc[1][2], sc[1][3]) : 0u;
      const uint32_t va = vb + (tw + (lane & 7) + ((lane >> 3) & 1) * 8) * PITCH + (lane >> 4) * 16;
#pragma unroll
      for (int np = 0; np < NBO / 2; ++np) {
        uint32_t b0, b1, b2, b3;
        la_ldsm_x4_trans(va + np * 32, b0, b1, b2, b3);
        float x[2][4];
#pragma unroll
        for (int q = 0; q < 2; ++q)
#pragma unroll
          for (int e = 0; e < 4; ++e) x[q][e] = e < 2 * RH ? o[2 * np + q][e < 2 * RH ? e : 0] * corr[e < 2 * RH ? e >> 1 : 0] : 0.0f;
        la_mma(x[0], pa0, pa1, pa2, pa3, b0, b1);
        la_mma(x[1], pa0, pa1, pa2, pa3, b2, b3);
#pragma unroll
        for (int q = 0; q < 2; ++q)
#pragma unroll
          for (int e = 0; e < 2 * RH; ++e) o[2 * np + q][e] = x[q][e];
      }
    }
    __syncthreads();   // the stage is overwritten by the copy issued in the next iteration
  }
  la_wait<0>();
  __syncthreads();
  // the four warps' states: [warp][head][max, sum, -, - | D]
  float* s_rec = reinterpret_cast<float*>(smem);
#pragma unroll
  for (int r = 0; r < RH; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    if (g8 + 8 * r < nh) {
      float* rec = s_rec + (w * nh + g8 + 8 * r) * REC;
      if (t4 == 0) {
        rec[0] = m[r];
        rec[1] = l[r];
      }
#pragma unroll
      for (int nb = 0; nb < NBO; ++nb) *reinterpret_cast<float2*>(rec + 4 + nb * 8 + 2 * t4) = make_float2(o[nb][2 * r], o[nb][2 * r + 1]);
    }
  }
  __syncthreads();
  const bf16* gate = a.g_col >= 0 ? row + a.g_col + h0 : nullptr;
  bf16* out = reinterpret_cast<bf16*>(a.out) + ((int64_t)b * sh.H + h0) * sh.vdim;
  const int rec_out = sh.dv + 4;
  float* part = a.part + (((int64_t)b * gridDim.y + blockIdx.y) * hp) * splits * rec_out;   // [head][split][record]
  for (int i = tid; i < nh * sh.dv; i += kGaThreads) {
    const int g = i / sh.dv, e = i % sh.dv;
    float mx = splits == 1 && a.sink ? a.sink[h0 + g] : -INFINITY;
#pragma unroll
    for (int q = 0; q < 4; ++q) mx = fmaxf(mx, s_rec[(q * nh + g) * REC]);
    float L = splits == 1 && a.sink ? expf(a.sink[h0 + g] - mx) : 0.0f, A = 0.0f;
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const float* rec = s_rec + (q * nh + g) * REC;
      const float c = rec[0] == -INFINITY ? 0.0f : expf(rec[0] - mx);
      L += rec[1] * c;
      A += rec[4 + e] * c;
    }
    if (splits == 1) {
      if (e < sh.vdim) out[g * sh.vdim + e] = from_f<bf16>((L > 0.0f ? A / L : 0.0f) * (gate ? head_gate(to_f<bf16>(gate[g])) : 1.0f));
    } else {
      float* pr = part + ((int64_t)g * splits + split) * rec_out;
      if (e == 0) {
        pr[0] = mx;
        pr[1] = L;
      }
      pr[4 + e] = A;
    }
  }
  if (splits == 1) return;
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    unsigned* cnt = a.counters + (int64_t)b * gridDim.y + blockIdx.y;
    const unsigned prev = atomicAdd(cnt, 1u);
    s_last = prev == (unsigned)splits - 1u;
    if (s_last) *cnt = 0u;
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  // weights of the splits, then four columns of one head per thread
  float* s_w = s_rec;   // [head][splits]
  for (int g = w; g < nh; g += kGaThreads / 32) {
    const float* pr = part + (int64_t)g * splits * rec_out;
    const float m0 = lane < splits ? __ldcg(pr + (int64_t)lane * rec_out) : -INFINITY, m1 = lane + 32 < splits ? __ldcg(pr + (int64_t)(lane + 32) * rec_out) : -INFINITY;
    const float l0 = lane < splits ? __ldcg(pr + (int64_t)lane * rec_out + 1) : 0.0f, l1 = lane + 32 < splits ? __ldcg(pr + (int64_t)(lane + 32) * rec_out + 1) : 0.0f;
    const float sink = a.sink ? a.sink[h0 + g] : -INFINITY;
    const float mx = fmaxf(sink, warp_max(fmaxf(m0, m1)));
    const float e0 = m0 == -INFINITY ? 0.0f : expf(m0 - mx), e1 = m1 == -INFINITY ? 0.0f : expf(m1 - mx);
    const float L = warp_sum(l0 * e0 + l1 * e1) + (a.sink ? expf(sink - mx) : 0.0f);
    const float f = (L > 0.0f ? 1.0f / L : 0.0f) * (gate ? head_gate(to_f<bf16>(gate[g])) : 1.0f);
    if (lane < splits) s_w[g * kGroupedMaxSplits + lane] = e0 * f;
    if (lane + 32 < splits) s_w[g * kGroupedMaxSplits + lane + 32] = e1 * f;
  }
  __syncthreads();
  const int quads = sh.dv / 4;
  for (int i = tid; i < nh * quads; i += kGaThreads) {
    const int g = i / quads, e = (i % quads) * 4;
    const float4* pr = reinterpret_cast<const float4*>(part + (int64_t)g * splits * rec_out + 4 + e);
    float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 8
    for (int q = 0; q < splits; ++q) {
      const float4 t = __ldcg(pr + (int64_t)q * (rec_out / 4));
      const float f = s_w[g * kGroupedMaxSplits + q];
      x.x = fmaf(f, t.x, x.x); x.y = fmaf(f, t.y, x.y); x.z = fmaf(f, t.z, x.z); x.w = fmaf(f, t.w, x.w);
    }
    const float xs[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (e + k < sh.vdim) out[g * sh.vdim + e + k] = from_f<bf16>(xs[k]);
  }
}

__global__ void expand_bias_f32_kernel(float* out, const float* table, const int* bucket, int n, int H) {
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n * H; i += gridDim.x * blockDim.x) out[i] = table[(int64_t)bucket[i % n] * H + i / n];
}
__global__ void expand_bias_bf16_kernel(float* out, const bf16* table, const int* bucket, int n, int H) {
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n * H; i += gridDim.x * blockDim.x) out[i] = to_f<bf16>(table[(int64_t)bucket[i % n] * H + i / n]);
}

// ---- host side -------------------------------------------------------------------------------------------------------------------
int launch_expand_bias(int device, int src_dtype, float* out, const void* table, const int* bucket, int n, int H, cudaStream_t s) {
  const int g = (int)std::min<int64_t>(((int64_t)n * H + 255) / 256, 4096);
  if (src_dtype == TSB200_F32) expand_bias_f32_kernel<<<g, 256, 0, s>>>(out, (const float*)table, bucket, n, H);
  else expand_bias_bf16_kernel<<<g, 256, 0, s>>>(out, (const bf16*)table, bucket, n, H);
  count_launch(device);
  return check_launch("expand_bias");
}

// staged row size that serves a shape; 0: none
static int grouped_tile(int dtype, const GroupedShape& a) {
  if (dtype != TSB200_BF16 || a.vdim % 2 != 0) return 0;
  const int n = a.dk > a.dv ? a.dk : a.dv;
  for (int d : {32, 64, 96, 128, 192, 256})
    if (n <= d) return d;
  return 0;
}
static int grouped_decode_heads(const GroupedShape& a) {   // query heads of a CTA
  const int group = a.H / a.G;
  return group < 16 ? group : 16;
}
int grouped_pick_splits(DeviceState* st, int dtype, const GroupedShape& a, int B, int T) {
  const int D = grouped_tile(dtype, a);
  if (!D) return 1;
  const int group = a.H / a.G, hp = grouped_decode_heads(a);
  const int64_t base = (int64_t)B * a.G * ((group + hp - 1) / hp);
  const int n = a.window > 0 ? std::min(T, a.window + a.keep_first) : T;
  // CTAs that run at a time; a split costs its keys, about two tiles for its start and three for its part in the merge (measured)
  const int64_t slots = (int64_t)st->sm_count * (D <= 64 ? 5 : D <= 96 ? 4 : D <= 128 ? 3 : D <= 192 ? 2 : 1);
  int best = 1;
  int64_t best_cost = 0;
  for (int s = 1; s <= std::min(kGroupedMaxSplits, (n + 127) / 128); ++s) {
    const int64_t cost = (base * s + slots - 1) / slots * ((n + s - 1) / s + (s > 1 ? 5 : 2) * kGaKeys);
    if (s == 1 || cost < best_cost) {
      best = s;
      best_cost = cost;
    }
  }
  return best;
}
int64_t grouped_part_elems(const GroupedShape& a, int B, int splits) {
  if (splits <= 1) return 0;
  const int group = a.H / a.G, hp = grouped_decode_heads(a);
  return (int64_t)B * a.G * ((group + hp - 1) / hp) * hp * splits * (a.dv + 4);
}

template <int D>
static int grouped_prefill_go(int device, const GroupedArgs& a, cudaStream_t s) {
  const GroupedShape& sh = a.shape;
  const int group = sh.H / sh.G, hp = group < 64 ? group : 64, chunks = (group + hp - 1) / hp, qt = 64 / hp;
  const int64_t bias_bytes = (int64_t)hp * sh.n_bias * 4;
  const int in_smem = sh.n_bias > 0 && bias_bytes <= 16 * 1024;
  const size_t smem = (size_t)kGaStages * GaTile<D>::stage + (in_smem ? (size_t)bias_bytes : 0);
  static bool done[kMaxDevices] = {};
  if (!done[device]) {
    TSB_CUDA(cudaFuncSetAttribute(grouped_prefill_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(kGaStages * GaTile<D>::stage + 16 * 1024)));
    done[device] = true;
  }
  TSB_CHECK((int64_t)sh.G * chunks <= 65535 && a.B <= 65535, "grouped attention: %d key/value heads of %d sequences are not supported", sh.G, a.B);
  TSB_CUDA(launch_k(grouped_prefill_kernel<D>, dim3((a.S + qt - 1) / qt, sh.G * chunks, a.B), dim3(kGaThreads), smem, s, a, hp, qt, in_smem));
  count_launch(device);
  return check_launch("grouped_prefill");
}
template <int D, int RH>
static int grouped_decode_go(int device, const GroupedArgs& a, int hp, cudaStream_t s) {
  const GroupedShape& sh = a.shape;
  const size_t smem = (size_t)kGaStages * GaTile<D>::stage + 8 * RH * GaTile<D>::pitch + 2 * D * 2;
  static bool done[kMaxDevices] = {};
  if (!done[device]) {
    TSB_CUDA(cudaFuncSetAttribute(grouped_decode_kernel<D, RH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    done[device] = true;
  }
  const int chunks = (sh.H / sh.G + hp - 1) / hp;
  TSB_CHECK((int64_t)sh.G * chunks <= 65535 && a.B <= 65535, "grouped attention: %d key/value heads of %d sequences are not supported", sh.G, a.B);
  TSB_CUDA(launch_k(grouped_decode_kernel<D, RH>, dim3(a.splits, sh.G * chunks, a.B), dim3(kGaThreads), smem, s, a, hp));
  count_launch(device);
  return check_launch("grouped_decode");
}

int launch_grouped_attention(int device, DeviceState* st, int dtype, const GroupedArgs& a, cudaStream_t s) {
  if (a.B == 0 || a.S == 0) return 1;
  const GroupedShape& sh = a.shape;
  TSB_CHECK(sh.G > 0 && sh.H % sh.G == 0, "grouped attention: %d heads do not share %d key/value heads", sh.H, sh.G);
  TSB_CHECK(a.state || a.T0 + a.S <= a.Tmax, "grouped attention: cache capacity exceeded (%d + %d > %d)", a.T0, a.S, a.Tmax);
  const int D = grouped_tile(dtype, sh);
  if (D && a.S == 1) {
    const int hp = grouped_decode_heads(sh);
    TSB_CHECK(a.splits >= 1 && a.splits <= kGroupedMaxSplits && grouped_part_elems(sh, a.B, a.splits) <= a.part_elems,
              "grouped attention: scratch too small for %d splits", a.splits);
#define TSB_GD(DD) case DD: return hp <= 8 ? grouped_decode_go<DD, 1>(device, a, hp, s) : grouped_decode_go<DD, 2>(device, a, hp, s)
    switch (D) {
      TSB_GD(32);
      TSB_GD(64);
      TSB_GD(96);
      TSB_GD(128);
      TSB_GD(192);
      TSB_GD(256);
    }
#undef TSB_GD
  }
  // queries normed into the scratch, keys and values appended
  {
    const int64_t units = (int64_t)a.B * a.S * (sh.H + (a.k_col >= 0 ? 2 * sh.G : 0));
    TSB_CHECK(units < (1LL << 31), "grouped attention: portions of %d tokens are not supported", a.B * a.S);
    const int g = (int)std::min<int64_t>((units + 7) / 8, (int64_t)st->sm_count * 16);
    const bool v4 = sh.dim % 4 == 0 && sh.vdim % 4 == 0 && a.q_stride % 4 == 0 && a.k_col % 4 == 0 && a.v_col % 4 == 0 && ((uintptr_t)a.qkv % 16) == 0;
    const bool v4s = v4 || (a.k_col < 0 && sh.dim % 4 == 0 && a.q_stride % 4 == 0 && ((uintptr_t)a.qkv % 16) == 0);
    if (dtype == TSB200_F32) TSB_CUDA(launch_k(v4s ? head_prep_kernel<float, 4> : head_prep_kernel<float, 1>, dim3(g), dim3(256), 0, s, a));
    else TSB_CUDA(launch_k(v4s ? head_prep_kernel<bf16, 4> : head_prep_kernel<bf16, 1>, dim3(g), dim3(256), 0, s, a));
    count_launch(device);
    TSB_TRY(check_launch("head_prep"));
  }
  switch (D) {
    case 32: return grouped_prefill_go<32>(device, a, s);
    case 64: return grouped_prefill_go<64>(device, a, s);
    case 96: return grouped_prefill_go<96>(device, a, s);
    case 128: return grouped_prefill_go<128>(device, a, s);
    case 192: return grouped_prefill_go<192>(device, a, s);
    case 256: return grouped_prefill_go<256>(device, a, s);
  }
  const size_t smem = ((size_t)sh.dk + sh.vdim + kGsimThreads + 32) * sizeof(float);
  TSB_CHECK(smem <= 48 * 1024, "grouped attention: heads of %d + %d values are not supported", sh.dim, sh.vdim);
  // rows go in the second grid dimension
  for (int64_t r0 = 0; r0 < (int64_t)a.B * a.S;) {
    // whole sequences per launch keep the row arithmetic; one launch unless there are more than 65535 rows
    const int64_t seqs = std::max<int64_t>(1, 65535 / a.S), b0 = r0 / a.S;
    GroupedArgs c = a;
    c.B = (int)std::min<int64_t>(seqs, a.B - b0);
    TSB_CHECK((int64_t)c.B * a.S <= 65535, "grouped attention: portions of %d tokens are not supported in this type", a.S);
    const int es = (int)dtype_size(dtype);
    TSB_CHECK(b0 == 0 || !a.state, "grouped attention: too many rows for one step");
    c.qkv = (const char*)a.qkv + r0 * a.q_stride * es;
    c.qn = (char*)a.qn + r0 * sh.H * sh.dk * es;
    c.out = (char*)a.out + r0 * sh.H * sh.vdim * es;
    c.cK = (char*)a.cK + b0 * sh.G * a.Tmax * sh.dk * es;
    c.cV = (char*)a.cV + b0 * sh.G * a.Tmax * sh.dv * es;
    const dim3 grid(sh.H, (unsigned)(c.B * a.S));
    if (dtype == TSB200_F32) TSB_CUDA(launch_k(grouped_simple_kernel<float>, grid, dim3(kGsimThreads), smem, s, c));
    else TSB_CUDA(launch_k(grouped_simple_kernel<bf16>, grid, dim3(kGsimThreads), smem, s, c));
    count_launch(device);
    TSB_TRY(check_launch("grouped_simple"));
    r0 += (int64_t)c.B * a.S;
  }
  return 1;
}

}  // namespace tsb
