// Matrix memory with exponential gates (the mLSTM recurrence): per head a matrix S [dim, vdim], a vector n [dim] and a running maximum m
// that keeps the exponentials in range.  With log gates i = cap tanh(z_i / cap) and f = logsigmoid(cap tanh(z_f / cap)):
//
//   m' = max(f + m, i);   S' = e^(f + m - m') S + e^(i - m') k v^T;   n' likewise with k;   (all zero before the first token)
//   o  = S'^T q / (max(|n' . q|, e^(-m')) + 1e-6),  q scaled by dim^(-1/2)
//   out = o / rms(o) * w * sigmoid(g)
//
// State of a sequence and layer: fp32, S [H][dim][vdim], n [H][dim], m [H].  Position 0 starts from zero, so a slot that is used again
// needs no clearing.
//
//   memory_step_kernel   token by token, a cluster of CTAs per (sequence, head) with the value columns shared out; the sum of squares of
//                        the norm crosses the cluster through distributed shared memory.  Decoding, short portions, fp32 models.
//   prompts (bf16), in chunks of 128 tokens, with F the running sum of f inside a chunk:
//   memory_gates_kernel  log gates, F and the running maximum of every token (a scan with (max, +))
//   memory_state_kernel  a tile of S per CTA, chunk by chunk in registers: S <- e^(F_C + m_0 - m_C) S + sum_s e^(F_C - F_s + i_s - m_C) k_s v_s^T
//                        on the warp-level tensor cores; leaves the state before every chunk in scratch
//   memory_out_kernel    64 tokens per CTA: inside the chunk (q_t . k_s) e^(F_t - F_s + i_s - m_t), before it e^(F_t + m_0 - m_t) S^T q,
//                        denominator, norm and output gate
// The chunk kernels keep fp32 quality on bf16 products: weighted values, scores and states enter as a sum of two bf16 numbers.
#include <algorithm>

#include "kernels.cuh"
#include "warp_tiles.cuh"

namespace tsb {

TSB_CHECKED_WORD(memory)
#ifndef TSB200_CHECKED
int chk_take_memory() { return 0; }
#endif

__device__ __forceinline__ float log_sigmoid(float z) { return z >= 0.0f ? -log1pf(expf(-z)) : z - log1pf(expf(z)); }
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

__device__ __forceinline__ void cluster_sync() {
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float cluster_read(const float* p, unsigned rank) {
  uint32_t a;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(la_smem(p)), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
  return v;
}

// ---- token by token ----------------------------------------------------------------------------------------------------------------
constexpr int kMsThreads = 256, kMsBatch = 8;

template <int V> struct MsVec;
template <> struct MsVec<1> {
  static __device__ __forceinline__ void load(const float* p, float* f) { f[0] = *p; }
  static __device__ __forceinline__ void store(float* p, const float* f) { *p = f[0]; }
};
template <> struct MsVec<4> {
  static __device__ __forceinline__ void load(const float* p, float* f) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    f[0] = t.x; f[1] = t.y; f[2] = t.z; f[3] = t.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};

// grid (cluster size, heads, sequences); the CTA of rank r has value columns [r * cw, min(vdim, (r + 1) * cw)), cw a multiple of V.
// Dynamic shared memory: q, k, n [dim each], v [cw], partial outputs [row groups][cw], 32 for sums.
template <typename T, int V>
__global__ void __launch_bounds__(kMsThreads) memory_step_kernel(MemoryArgs a, int cw) {
  extern __shared__ __align__(16) float s_mem[];
  __shared__ float s_sq[2];
  const MemoryShape& sh = a.shape;
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, rank = blockIdx.x, ranks = gridDim.x, h = blockIdx.y, b = blockIdx.z;
  const int dim = sh.dim, c0 = rank * cw, nc = min(cw, sh.vdim - c0);   // every rank has columns
  const int tpr = cw / V, groups = kMsThreads / tpr;                    // threads per matrix row, rows at a time
  float *s_q = s_mem, *s_k = s_q + dim, *s_n = s_k + dim, *s_v = s_n + dim, *s_o = s_v + cw, *s_red = s_o + groups * cw;
  const int T0 = state_len(a.step_state, b, a.T0);
  const int n_tok = a.lens ? min(max(a.lens[b], 1), a.S) : a.S;
  const bool still = a.stop_fin && a.step_state && a.step_state[kStateRagged] != 0 && a.ids[b] == 0;
  float* st = a.state + (int64_t)b * memory_state_floats(sh);
  float* S = st + (int64_t)h * dim * sh.vdim;
  float* gn = st + (int64_t)sh.H * dim * sh.vdim + (int64_t)h * dim;
  float* gm = st + (int64_t)sh.H * dim * sh.vdim + (int64_t)sh.H * dim + h;
  float m = T0 > 0 ? *gm : 0.0f;
  for (int i = tid; i < dim; i += kMsThreads) s_n[i] = T0 > 0 ? gn[i] : 0.0f;
  const float qs = 1.0f / sqrtf((float)dim);
  const int grp = tid / tpr, col = (tid % tpr) * V;
  const bool mine = grp < groups && col < nc;   // nc is a multiple of V
  const int64_t qk = (int64_t)sh.H * dim, vg = (int64_t)sh.H * sh.vdim;

  for (int t = 0; t < n_tok; ++t) {
    const int64_t row = (int64_t)b * a.S + t;
    const T* x = reinterpret_cast<const T*>(a.x) + row * a.stride;
    const float gi = soft_cap(a.gates[row * 2 * sh.H + h], sh.cap);
    const float gf = log_sigmoid(soft_cap(a.gates[row * 2 * sh.H + sh.H + h], sh.cap));
    const float mn = fmaxf(gf + m, gi), keep = expf(gf + m - mn), add = expf(gi - mn);
    m = mn;
    __syncthreads();   // the previous token's vectors have been read
    for (int i = tid; i < dim; i += kMsThreads) {
      s_q[i] = to_f<T>(x[(int64_t)h * dim + i]) * qs;
      s_k[i] = to_f<T>(x[qk + (int64_t)h * dim + i]);
    }
    for (int i = tid; i < nc; i += kMsThreads) s_v[i] = to_f<T>(x[2 * qk + (int64_t)h * sh.vdim + c0 + i]);
    __syncthreads();
    float dot = 0.0f;
    for (int i = tid; i < dim; i += kMsThreads) {
      const float nn = keep * s_n[i] + add * s_k[i];
      s_n[i] = nn;
      dot = fmaf(nn, s_q[i], dot);
    }
    if (mine) {
      float acc[V], v[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {
        acc[e] = 0.0f;
        v[e] = s_v[col + e] * add;
      }
      float* base = S + c0 + col;
      const bool zero = T0 + t == 0;
      for (int r0 = grp; r0 < dim; r0 += groups * kMsBatch) {
        float s[kMsBatch][V];
#pragma unroll
        for (int q = 0; q < kMsBatch; ++q) {
          const int r = r0 + q * groups;
#pragma unroll
          for (int e = 0; e < V; ++e) s[q][e] = 0.0f;
          if (r < dim && !zero) MsVec<V>::load(base + (int64_t)r * sh.vdim, s[q]);
        }
#pragma unroll
        for (int q = 0; q < kMsBatch; ++q) {
          const int r = r0 + q * groups;
          if (r >= dim) break;
          const float kk = s_k[r], qq = s_q[r];
#pragma unroll
          for (int e = 0; e < V; ++e) {
            s[q][e] = fmaf(v[e], kk, keep * s[q][e]);
            acc[e] = fmaf(s[q][e], qq, acc[e]);
          }
          if (!still) MsVec<V>::store(base + (int64_t)r * sh.vdim, s[q]);
        }
      }
#pragma unroll
      for (int e = 0; e < V; ++e) s_o[grp * cw + col + e] = acc[e];
    }
    dot = block_sum(dot, s_red);   // its barriers also publish s_o
    const float inv_den = 1.0f / (fmaxf(fabsf(dot), expf(-m)) + 1e-6f);
    float sq = 0.0f;
    for (int c = tid; c < nc; c += kMsThreads) {
      float o = 0.0f;
      for (int q = 0; q < groups; ++q) o += s_o[q * cw + c];
      o *= inv_den;
      sq = fmaf(o, o, sq);
      s_v[c] = o;
    }
    sq = block_sum(sq, s_red);
    if (ranks > 1) {
      if (tid == 0) s_sq[t & 1] = sq;
      cluster_sync();
      sq = 0.0f;
      for (int q = 0; q < ranks; ++q) sq += cluster_read(&s_sq[t & 1], q);
    }
    const float r = 1.0f / sqrtf(sq / (float)sh.vdim + sh.eps);
    for (int c = tid; c < nc; c += kMsThreads) {
      const int64_t e = (int64_t)h * sh.vdim + c0 + c;
      const float g = to_f<T>(x[2 * qk + vg + e]);
      reinterpret_cast<T*>(a.out)[row * vg + e] = from_f<T>(s_v[c] * r * to_f<T>(reinterpret_cast<const T*>(a.norm_w)[e]) / (1.0f + expf(-g)));
    }
  }
  // every rank has read n and m: the first cluster barrier lies behind
  if (rank == 0 && !still) {
    for (int i = tid; i < dim; i += kMsThreads) gn[i] = s_n[i];
    if (tid == 0) *gm = m;
  }
  if (ranks > 1) cluster_sync();   // no CTA leaves while another reads its sum
}

// ---- chunks ------------------------------------------------------------------------------------------------------------------------
constexpr int kMcTokens = 128;      // tokens per chunk
constexpr int kMcTile = 64;         // state tile, value slice, rows of an output CTA
constexpr int kMcPitch = kMcTile * 2 + 16;
constexpr int kMcMaxDim = 256;
constexpr int kMgThreads = 1024;

struct MemoryChunks {               // scratch of the chunk kernels
  float *F, *I, *M;                 // [B * H][chunks * 128]: sum of f inside the chunk, i, running maximum
  float* m0;                        // [B * H] running maximum before the portion
  float* n0;                        // [B * H][chunks][dim] state vector before every chunk
  bf16 *hi, *lo;                    // [B * H][chunks][dim][vdim] state before every chunk, as a sum of two numbers
  int chunks;
};
// a pair of values as the sum of two bf16 pairs
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = Pair16<bf16>::put(a, b);
  const float2 h = Pair16<bf16>::get(hi);
  lo = Pair16<bf16>::put(a - h.x, b - h.y);
}

__global__ void __launch_bounds__(kMgThreads) memory_gates_kernel(MemoryArgs a, MemoryChunks ck) {
  __shared__ float s_a[32], s_b[32];
  const MemoryShape& sh = a.shape;
  const int bh = blockIdx.x, b = bh / sh.H, h = bh % sh.H, tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
  const int T0 = state_len(a.step_state, b, a.T0);
  const int n_tok = a.lens ? min(max(a.lens[b], 1), a.S) : a.S, padded = ck.chunks * kMcTokens;
  float* gm = a.state + (int64_t)b * memory_state_floats(sh) + (int64_t)sh.H * sh.dim * sh.vdim + (int64_t)sh.H * sh.dim + h;
  float carry = T0 > 0 ? *gm : 0.0f;
  __syncthreads();
  if (tid == 0) ck.m0[bh] = carry;
  for (int t0 = 0; t0 < padded; t0 += kMgThreads) {
    const int t = t0 + tid;
    float gi = -INFINITY, gf = 0.0f;   // tokens beyond the end change nothing
    if (t < n_tok) {
      const int64_t row = (int64_t)b * a.S + t;
      gi = soft_cap(a.gates[row * 2 * sh.H + h], sh.cap);
      gf = log_sigmoid(soft_cap(a.gates[row * 2 * sh.H + sh.H + h], sh.cap));
    }
    // (A, B) of a range of tokens: m after it = max(A + m before it, B)
    float A = gf, B = gi;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pa = __shfl_up_sync(0xffffffffu, A, o), pb = __shfl_up_sync(0xffffffffu, B, o);
      if (lane >= o) {
        B = fmaxf(pb + A, B);
        A += pa;
      }
    }
    __syncthreads();
    if (lane == 31) {
      s_a[w] = A;
      s_b[w] = B;
    }
    __syncthreads();
    float F = A, m = carry;
    for (int q = w & ~3; q < w; ++q) F += s_a[q];          // four warps to a chunk
    for (int q = 0; q < w; ++q) m = fmaxf(s_a[q] + m, s_b[q]);
    m = fmaxf(A + m, B);
    for (int q = 0; q < 32; ++q) carry = fmaxf(s_a[q] + carry, s_b[q]);
    if (t < padded) {
      const int64_t at = (int64_t)bh * padded + t;
      ck.F[at] = F;
      ck.I[at] = gi;
      ck.M[at] = m;
    }
  }
  if (tid == 0) *gm = carry;
}

// grid (value tiles, key tiles, B * H), 4 warps of 16 matrix rows; keys, values and gate sums of a chunk are copied one chunk ahead
struct McStage {                    // shared memory of memory_state_kernel
  unsigned char k[2][kMcTokens * kMcPitch];
  unsigned char v[2][kMcTokens * kMcPitch];   // becomes the upper part of the weighted values
  unsigned char lo[kMcTokens * kMcPitch];
  float F[2][kMcTokens], I[2][kMcTokens];
};
__global__ void __launch_bounds__(128) memory_state_kernel(MemoryArgs a, MemoryChunks ck) {
  extern __shared__ __align__(128) unsigned char smem[];
  McStage& sm = *reinterpret_cast<McStage*>(smem);
  __shared__ float s_w[kMcTokens];
  const MemoryShape& sh = a.shape;
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
  const int v0 = blockIdx.x * kMcTile, d0 = blockIdx.y * kMcTile, bh = blockIdx.z, b = bh / sh.H, h = bh % sh.H;
  const int nv = min(kMcTile, sh.vdim - v0), nd = min(kMcTile, sh.dim - d0);
  const int T0 = state_len(a.step_state, b, a.T0), padded = ck.chunks * kMcTokens;
  float* st = a.state + (int64_t)b * memory_state_floats(sh);
  float* S = st + (int64_t)h * sh.dim * sh.vdim;
  float* gn = st + (int64_t)sh.H * sh.dim * sh.vdim + (int64_t)h * sh.dim;
  const int64_t qk = (int64_t)sh.H * sh.dim;
  const bf16* x0 = reinterpret_cast<const bf16*>(a.x) + (int64_t)b * a.S * a.stride;
  auto issue = [&](int c) {
    if (c < ck.chunks) {
      const uint32_t dk = la_smem(sm.k[c & 1]), dv = la_smem(sm.v[c & 1]);
      for (int v = tid; v < kMcTokens * 8; v += 128) {   // 8 units of 16 bytes per row
        const int r = v >> 3, u = v & 7, t = c * kMcTokens + r;
        const bool lk = t < a.S && u * 8 < nd, lv = t < a.S && u * 8 < nv;
        const bf16* xr = x0 + (int64_t)min(t, a.S - 1) * a.stride;
        la_cp16(dk + r * kMcPitch + u * 16, lk ? xr + qk + (int64_t)h * sh.dim + d0 + u * 8 : xr, lk);
        la_cp16(dv + r * kMcPitch + u * 16, lv ? xr + 2 * qk + (int64_t)h * sh.vdim + v0 + u * 8 : xr, lv);
      }
      if (tid < 64) {
        const int64_t at = (int64_t)bh * padded + c * kMcTokens + (tid & 31) * 4;
        la_cp16(la_smem(tid < 32 ? &sm.F[c & 1][tid * 4] : &sm.I[c & 1][(tid & 31) * 4]), (tid < 32 ? ck.F : ck.I) + at);
      }
    }
    la_commit();
  };
  issue(0);
  float s[8][4], nvec = 0.0f;
#pragma unroll
  for (int nb = 0; nb < 8; ++nb)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = w * 16 + g8 + (e >> 1) * 8, c = nb * 8 + 2 * t4 + (e & 1);
      s[nb][e] = T0 > 0 && r < nd && c < nv ? S[(int64_t)(d0 + r) * sh.vdim + v0 + c] : 0.0f;
    }
  const bool vec = blockIdx.x == 0 && tid < nd;   // one element of n per thread of the first value tile
  if (vec && T0 > 0) nvec = gn[d0 + tid];
  float m0 = ck.m0[bh], m_next = ck.M[(int64_t)bh * padded + kMcTokens - 1];
  for (int c = 0; c < ck.chunks; ++c) {
    issue(c + 1);
    const float mC = m_next;
    if (c + 1 < ck.chunks) m_next = ck.M[(int64_t)bh * padded + (c + 1) * kMcTokens + kMcTokens - 1];
    // the state before the chunk
    const int64_t plane = ((int64_t)bh * ck.chunks + c) * sh.dim * sh.vdim;
#pragma unroll
    for (int nb = 0; nb < 8; ++nb)
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const int r = w * 16 + g8 + q * 8, cc = nb * 8 + 2 * t4;
        if (r < nd && cc < nv) {
          uint32_t hi, lo;
          split_pair(s[nb][2 * q], s[nb][2 * q + 1], hi, lo);
          const int64_t at = plane + (int64_t)(d0 + r) * sh.vdim + v0 + cc;
          *reinterpret_cast<uint32_t*>(ck.hi + at) = hi;
          *reinterpret_cast<uint32_t*>(ck.lo + at) = lo;
        }
      }
    if (vec) ck.n0[((int64_t)bh * ck.chunks + c) * sh.dim + d0 + tid] = nvec;
    la_wait<1>();
    __syncthreads();
    const float *F = sm.F[c & 1], FC = F[kMcTokens - 1];
    const float keep = expf(FC + m0 - mC);
    s_w[tid] = expf(FC - F[tid] + sm.I[c & 1][tid] - mC);
    __syncthreads();
    for (int v = tid; v < kMcTokens * 8; v += 128) {   // values times their weight, in two parts
      const int r = v >> 3, at = r * kMcPitch + (v & 7) * 16;
      const uint4 in = *reinterpret_cast<const uint4*>(sm.v[c & 1] + at);
      uint4 hi, lo;
      const float wt = s_w[r];
      const uint32_t* pi = &in.x;
      uint32_t *ph = &hi.x, *pl = &lo.x;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = Pair16<bf16>::get(pi[e]);
        split_pair(f.x * wt, f.y * wt, ph[e], pl[e]);
      }
      *reinterpret_cast<uint4*>(sm.v[c & 1] + at) = hi;
      *reinterpret_cast<uint4*>(sm.lo + at) = lo;
    }
    __syncthreads();
#pragma unroll
    for (int nb = 0; nb < 8; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[nb][e] *= keep;
    // S += K^T V: rows of the product are key elements (fragments of K transposed), the sum runs over tokens
    const uint32_t ka = la_smem(sm.k[c & 1]) + ((lane & 7) + ((lane >> 4) & 1) * 8) * kMcPitch + (w * 16 + ((lane >> 3) & 1) * 8) * 2;
    const uint32_t vrow = ((lane & 7) + ((lane >> 3) & 1) * 8) * kMcPitch + (lane >> 4) * 16;
    const uint32_t va = la_smem(sm.v[c & 1]) + vrow, vl = la_smem(sm.lo) + vrow;
#pragma unroll
    for (int ks = 0; ks < kMcTokens / 16; ++ks) {
      uint32_t a0, a1, a2, a3;
      la_ldsm_x4_trans(ka + ks * 16 * kMcPitch, a0, a1, a2, a3);
#pragma unroll
      for (int part = 0; part < 2; ++part) {   // eight independent sums side by side
        uint32_t b[4][4];
#pragma unroll
        for (int np = 0; np < 4; ++np) la_ldsm_x4_trans((part ? vl : va) + ks * 16 * kMcPitch + np * 32, b[np][0], b[np][1], b[np][2], b[np][3]);
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          la_mma(s[2 * np], a0, a1, a2, a3, b[np][0], b[np][1]);
          la_mma(s[2 * np + 1], a0, a1, a2, a3, b[np][2], b[np][3]);
        }
      }
    }
    if (vec) {
      float d = 0.0f;
#pragma unroll 8
      for (int r = 0; r < kMcTokens; ++r) d = fmaf(s_w[r], to_f<bf16>(*reinterpret_cast<const bf16*>(sm.k[c & 1] + r * kMcPitch + tid * 2)), d);
      nvec = keep * nvec + d;
    }
    m0 = mC;
    __syncthreads();   // the next copy overwrites this chunk's stage
  }
  la_wait<0>();
#pragma unroll
  for (int nb = 0; nb < 8; ++nb)
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const int r = w * 16 + g8 + q * 8, c = nb * 8 + 2 * t4;
      if (r < nd && c < nv) *reinterpret_cast<float2*>(S + (int64_t)(d0 + r) * sh.vdim + v0 + c) = make_float2(s[nb][2 * q], s[nb][2 * q + 1]);
    }
  if (vec) gn[d0 + tid] = nvec;
}

// grid (tiles of 64 tokens, heads, sequences), 4 warps of 16 tokens.  Shared memory: q [64] rows; gated outputs [64] rows of vdim and 16
// bytes; then k [64] rows, or a value slice [128] and the two planes of a state slice [dim].  Rows of q and k hold dim elements rounded up to
// 16 (zero beyond) and 16 bytes.
__global__ void __launch_bounds__(128) memory_out_kernel(MemoryArgs a, MemoryChunks ck) {
  extern __shared__ __align__(128) unsigned char smem[];
  __shared__ float s_F[kMcTokens], s_key[kMcTokens], s_nq[kMcTile], s_n[kMcMaxDim];   // s_key: (i - F) in powers of two
  const MemoryShape& sh = a.shape;
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
  const int t0 = blockIdx.x * kMcTile, h = blockIdx.y, b = blockIdx.z, bh = b * sh.H + h;
  const int c = t0 / kMcTokens, cb = c * kMcTokens, padded = ck.chunks * kMcTokens;
  const int n_keys = t0 - cb + kMcTile;                       // 64 or 128, the tile's own tokens last
  const int dp = (sh.dim + 15) / 16 * 16, pitch = dp * 2 + 16, du = dp / 8;
  const int opitch = sh.vdim * 2 + 16;
  unsigned char* s_out = smem + kMcTile * pitch;
  const uint32_t sq = la_smem(smem), sk = la_smem(s_out) + kMcTile * opitch;
  const uint32_t sv = sk, sh_hi = sv + kMcTokens * kMcPitch, sh_lo = sh_hi + dp * kMcPitch;
  const int64_t qk = (int64_t)sh.H * sh.dim, vg = (int64_t)sh.H * sh.vdim;
  const bf16* x0 = reinterpret_cast<const bf16*>(a.x) + (int64_t)b * a.S * a.stride;
  auto rows = [&](uint32_t dst, int first, int64_t col) {     // 64 rows of q or k
    for (int r = w; r < kMcTile; r += 4)
      for (int u = lane; u < du; u += 32) {
        const int t = first + r;
        const bool live = t < a.S && u * 8 < sh.dim;
        la_cp16(dst + r * pitch + u * 16, live ? x0 + (int64_t)t * a.stride + col + (int64_t)h * sh.dim + u * 8 : x0, live);
      }
    la_commit();
  };
  rows(sq, t0, 0);
  rows(sk, cb, qk);
  s_F[tid] = ck.F[(int64_t)bh * padded + cb + tid];
  s_key[tid] = (ck.I[(int64_t)bh * padded + cb + tid] - s_F[tid]) * kLog2e;
  for (int i = tid; i < sh.dim; i += 128) s_n[i] = ck.n0[((int64_t)bh * ck.chunks + c) * sh.dim + i];
  const float m0 = c > 0 ? ck.M[(int64_t)bh * padded + cb - 1] : ck.m0[bh];
  const int rA = w * 16 + g8, off = t0 - cb;
  float mt[2], query[2], inter[2];   // query: (F - m) in powers of two
  const float qs = 1.0f / sqrtf((float)sh.dim);
  la_wait<0>();
  __syncthreads();
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    mt[q] = ck.M[(int64_t)bh * padded + t0 + rA + q * 8];
    const float ft = s_F[off + rA + q * 8];
    query[q] = (ft - mt[q]) * kLog2e;
    inter[q] = expf(ft + m0 - mt[q]) * qs;
  }
  {   // n . q of every row: two threads per row
    const bf16* qr = reinterpret_cast<const bf16*>(smem + (tid >> 1) * pitch);
    float d = 0.0f;
#pragma unroll 4
    for (int i = (tid & 1); i < sh.dim; i += 2) d = fmaf(s_n[i], to_f<bf16>(qr[i]), d);
    d += __shfl_xor_sync(0xffffffffu, d, 1);
    if ((tid & 1) == 0) s_nq[tid >> 1] = d;
  }
  // weights of the chunk's keys up to each row, as operands of the second product
  uint32_t ph[8][4], pl[8][4];
  float rs[2] = {0.0f, 0.0f};
  const uint32_t qa = sq + (w * 16 + (lane & 15)) * pitch + (lane >> 4) * 16;
#pragma unroll
  for (int kt = 0; kt < 2; ++kt) {
    if (kt * kMcTile < n_keys) {
      if (kt > 0) {
        __syncthreads();
        rows(sk, cb + kMcTile, qk);
        la_wait<0>();
        __syncthreads();
      }
      float sc[8][4];
#pragma unroll
      for (int nb = 0; nb < 8; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[nb][e] = 0.0f;
      const uint32_t ka = sk + ((lane & 7) + (lane >> 4) * 8) * pitch + ((lane >> 3) & 1) * 16;
      for (int ks = 0; ks < dp / 16; ++ks) {
        uint32_t a0, a1, a2, a3;
        la_ldsm_x4(qa + ks * 32, a0, a1, a2, a3);
#pragma unroll
        for (int np = 0; np < 4; ++np) {   // two blocks of 8 keys
          uint32_t b0, b1, b2, b3;
          la_ldsm_x4(ka + np * 16 * pitch + ks * 32, b0, b1, b2, b3);
          la_mma(sc[2 * np], a0, a1, a2, a3, b0, b1);
          la_mma(sc[2 * np + 1], a0, a1, a2, a3, b2, b3);
        }
      }
#pragma unroll
      for (int nb = 0; nb < 8; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int q = e >> 1, key = kt * kMcTile + nb * 8 + 2 * t4 + (e & 1);
          const float p = key <= off + rA + q * 8 ? sc[nb][e] * qs * exp2_fast(query[q] + s_key[key]) : 0.0f;
          sc[nb][e] = p;
          rs[q] += p;
        }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float* p = &sc[2 * kk + (e >> 1)][2 * (e & 1)];
          split_pair(p[0], p[1], ph[kt * 4 + kk][e], pl[kt * 4 + kk][e]);
        }
    } else {
#pragma unroll
      for (int kk = 0; kk < 4; ++kk)
#pragma unroll
        for (int e = 0; e < 4; ++e) ph[kt * 4 + kk][e] = pl[kt * 4 + kk][e] = 0u;
    }
  }
  __syncthreads();
  float inv_den[2], sq_sum[2] = {0.0f, 0.0f};
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    rs[q] += __shfl_xor_sync(0xffffffffu, rs[q], 1);
    rs[q] += __shfl_xor_sync(0xffffffffu, rs[q], 2);
    inv_den[q] = 1.0f / (fmaxf(fabsf(rs[q] + inter[q] * s_nq[rA + q * 8]), expf(-mt[q])) + 1e-6f);
  }
  const int64_t plane = ((int64_t)bh * ck.chunks + c) * sh.dim * sh.vdim;
  for (int v0 = 0; v0 < sh.vdim; v0 += kMcTile) {
    const int nv = min(kMcTile, sh.vdim - v0);
    if (v0 > 0) __syncthreads();
    for (int v = tid; v < n_keys * 8; v += 128) {
      const int r = v >> 3, u = v & 7, t = cb + r;
      const bool live = t < a.S && u * 8 < nv;
      la_cp16(sv + r * kMcPitch + u * 16, live ? x0 + (int64_t)t * a.stride + 2 * qk + (int64_t)h * sh.vdim + v0 + u * 8 : x0, live);
    }
    for (int v = tid; v < dp * 8; v += 128) {
      const int r = v >> 3, u = v & 7;
      const bool live = r < sh.dim && u * 8 < nv;
      const int64_t at = live ? plane + (int64_t)r * sh.vdim + v0 + u * 8 : 0;
      la_cp16(sh_hi + r * kMcPitch + u * 16, ck.hi + at, live);
      la_cp16(sh_lo + r * kMcPitch + u * 16, ck.lo + at, live);
    }
    la_commit();
    uint32_t gate[8][2], nw[8];   // output gates and norm weights of this thread's values, requested while the slice travels
#pragma unroll
    for (int nb = 0; nb < 8; ++nb) {
      const int cc = v0 + nb * 8 + 2 * t4;
      nw[nb] = cc < sh.vdim ? *reinterpret_cast<const uint32_t*>(reinterpret_cast<const bf16*>(a.norm_w) + (int64_t)h * sh.vdim + cc) : 0u;
#pragma unroll
      for (int q = 0; q < 2; ++q)
        gate[nb][q] = cc < sh.vdim && t0 + rA + q * 8 < a.S
                          ? *reinterpret_cast<const uint32_t*>(x0 + (int64_t)(t0 + rA + q * 8) * a.stride + 2 * qk + vg + (int64_t)h * sh.vdim + cc) : 0u;
    }
    la_wait<0>();
    __syncthreads();
    float o[8][4];
#pragma unroll
    for (int nb = 0; nb < 8; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[nb][e] = 0.0f;
    const uint32_t vrow = ((lane & 7) + ((lane >> 3) & 1) * 8) * kMcPitch + (lane >> 4) * 16;
    for (int ks = 0; ks < dp / 16; ++ks) {
      uint32_t a0, a1, a2, a3;
      la_ldsm_x4(qa + ks * 32, a0, a1, a2, a3);
#pragma unroll
      for (int part = 0; part < 2; ++part) {
        uint32_t b[4][4];
#pragma unroll
        for (int np = 0; np < 4; ++np) la_ldsm_x4_trans((part ? sh_lo : sh_hi) + vrow + ks * 16 * kMcPitch + np * 32, b[np][0], b[np][1], b[np][2], b[np][3]);
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          la_mma(o[2 * np], a0, a1, a2, a3, b[np][0], b[np][1]);
          la_mma(o[2 * np + 1], a0, a1, a2, a3, b[np][2], b[np][3]);
        }
      }
    }
#pragma unroll
    for (int nb = 0; nb < 8; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[nb][e] *= inter[e >> 1];
#pragma unroll
    for (int kk = 0; kk < 8; ++kk) {
      if (kk * 16 >= n_keys) break;
      uint32_t b[4][4];
#pragma unroll
      for (int np = 0; np < 4; ++np) la_ldsm_x4_trans(sv + vrow + kk * 16 * kMcPitch + np * 32, b[np][0], b[np][1], b[np][2], b[np][3]);
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        la_mma(o[2 * np], ph[kk][0], ph[kk][1], ph[kk][2], ph[kk][3], b[np][0], b[np][1]);
        la_mma(o[2 * np + 1], ph[kk][0], ph[kk][1], ph[kk][2], ph[kk][3], b[np][2], b[np][3]);
      }
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        la_mma(o[2 * np], pl[kk][0], pl[kk][1], pl[kk][2], pl[kk][3], b[np][0], b[np][1]);
        la_mma(o[2 * np + 1], pl[kk][0], pl[kk][1], pl[kk][2], pl[kk][3], b[np][2], b[np][3]);
      }
    }
#pragma unroll
    for (int nb = 0; nb < 8; ++nb)
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const float u0 = o[nb][2 * q] * inv_den[q], u1 = o[nb][2 * q + 1] * inv_den[q];
        sq_sum[q] += u0 * u0 + u1 * u1;   // columns beyond the slice are zero
        const int cc = nb * 8 + 2 * t4;
        const float2 g = Pair16<bf16>::get(gate[nb][q]), wt = Pair16<bf16>::get(nw[nb]);
        if (cc < nv)
          *reinterpret_cast<uint32_t*>(s_out + (rA + q * 8) * opitch + (v0 + cc) * 2) = Pair16<bf16>::put(__fdividef(u0 * wt.x, 1.0f + exp2_fast(-g.x * kLog2e)), __fdividef(u1 * wt.y, 1.0f + exp2_fast(-g.y * kLog2e)));
      }
  }
  // the norm's factor of every row; rows leave in 16-byte units
  float f[2];
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    sq_sum[q] += __shfl_xor_sync(0xffffffffu, sq_sum[q], 1);
    sq_sum[q] += __shfl_xor_sync(0xffffffffu, sq_sum[q], 2);
    f[q] = 1.0f / sqrtf(sq_sum[q] / (float)sh.vdim + sh.eps);
  }
  __syncwarp();
  bf16* out = reinterpret_cast<bf16*>(a.out) + ((int64_t)b * a.S + t0) * vg + (int64_t)h * sh.vdim;
#pragma unroll
  for (int r = 0; r < 16; ++r) {
    const float fr = __shfl_sync(0xffffffffu, f[r >> 3], (r & 7) * 4);
    if (t0 + w * 16 + r >= a.S) break;
    for (int u = lane; u < sh.vdim / 8; u += 32) {
      uint4 v = *reinterpret_cast<const uint4*>(s_out + (w * 16 + r) * opitch + u * 16);
      uint32_t* pv = &v.x;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 x = Pair16<bf16>::get(pv[e]);
        pv[e] = Pair16<bf16>::put(x.x * fr, x.y * fr);
      }
      *reinterpret_cast<uint4*>(out + (int64_t)(w * 16 + r) * vg + u * 8) = v;
    }
  }
}

// ---- host side -------------------------------------------------------------------------------------------------------------------
constexpr int kMemoryChunkMin = 32;   // shorter portions go token by token
constexpr size_t kMemorySmem = 220 * 1024;
static size_t memory_out_smem(const MemoryShape& a) {
  const int dp = (a.dim + 15) / 16 * 16;
  const size_t q = (size_t)kMcTile * (dp * 2 + 16);
  return q + (size_t)kMcTile * (a.vdim * 2 + 16) + std::max<size_t>(q, (size_t)(kMcTokens + 2 * dp) * kMcPitch);
}
static bool memory_chunked(int dtype, const MemoryShape& a, int S) {
  return dtype == TSB200_BF16 && S >= kMemoryChunkMin && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= kMcMaxDim && memory_out_smem(a) <= kMemorySmem;
}
static int64_t align16(int64_t n) { return (n + 255) / 256 * 256; }
static int64_t memory_layout(const MemoryShape& a, int B, int S, char* base, MemoryChunks* ck) {
  const int64_t bh = (int64_t)B * a.H, chunks = (S + kMcTokens - 1) / kMcTokens, tok = align16(bh * chunks * kMcTokens * 4), m0 = align16(bh * 4);
  const int64_t n0 = align16(bh * chunks * a.dim * 4), st = align16(bh * chunks * a.dim * a.vdim * 2);
  if (ck) {
    ck->chunks = (int)chunks;
    ck->F = (float*)base;
    ck->I = (float*)(base + tok);
    ck->M = (float*)(base + 2 * tok);
    ck->m0 = (float*)(base + 3 * tok);
    ck->n0 = (float*)(base + 3 * tok + m0);
    ck->hi = (bf16*)(base + 3 * tok + m0 + n0);
    ck->lo = (bf16*)(base + 3 * tok + m0 + n0 + st);
  }
  return 3 * tok + m0 + n0 + 2 * st;
}
int64_t memory_scratch_bytes(int dtype, const MemoryShape& a, int B, int S) { return memory_chunked(dtype, a, S) ? memory_layout(a, B, S, nullptr, nullptr) : 0; }

template <typename T, int V>
static int memory_step_go(int device, const MemoryArgs& a, int ranks, int cw, size_t smem, cudaStream_t s) {
  static bool done[kMaxDevices] = {};
  if (!done[device]) {
    TSB_CUDA(cudaFuncSetAttribute(memory_step_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    done[device] = true;
  }
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3(ranks, a.shape.H, a.B);
  cfg.blockDim = dim3(kMsThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute at[2];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = (unsigned)ranks;
  at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
  at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  at[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = at;
  cfg.numAttrs = pdl_enabled() ? 2 : 1;
  TSB_CUDA(cudaLaunchKernelEx(&cfg, memory_step_kernel<T, V>, a, cw));
  count_launch(device);
  return check_launch("memory_step");
}

int launch_matrix_memory(int device, DeviceState* st, int dtype, const MemoryArgs& a, cudaStream_t s) {
  if (a.B == 0 || a.S == 0) return 1;
  const MemoryShape& sh = a.shape;
  TSB_CHECK(a.B <= 65535 && sh.H <= 65535, "matrix memory: %d heads of %d sequences are not supported", sh.H, a.B);
  if (!a.step_state && memory_chunked(dtype, sh, a.S) && a.stride % 8 == 0 && ((uintptr_t)a.x % 16) == 0 && ((uintptr_t)a.state % 16) == 0) {
    MemoryChunks ck;
    TSB_CHECK(memory_layout(sh, a.B, a.S, (char*)a.scratch, &ck) <= a.scratch_bytes, "matrix memory: scratch too small for %d tokens", a.B * a.S);
    const size_t s1 = sizeof(McStage), s2 = memory_out_smem(sh);
    static bool done[kMaxDevices] = {};
    if (!done[device]) {
      TSB_CUDA(cudaFuncSetAttribute(memory_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(McStage)));
      TSB_CUDA(cudaFuncSetAttribute(memory_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMemorySmem));
      done[device] = true;
    }
    TSB_CHECK((int64_t)a.B * sh.H <= 65535, "matrix memory: %d heads of %d sequences are not supported", sh.H, a.B);
    memory_gates_kernel<<<a.B * sh.H, kMgThreads, 0, s>>>(a, ck);
    memory_state_kernel<<<dim3((sh.vdim + kMcTile - 1) / kMcTile, (sh.dim + kMcTile - 1) / kMcTile, a.B * sh.H), 128, s1, s>>>(a, ck);
    memory_out_kernel<<<dim3((a.S + kMcTile - 1) / kMcTile, sh.H, a.B), 128, s2, s>>>(a, ck);
    count_launch(device, 3);
    return check_launch("matrix_memory");
  }
  // columns of a CTA: enough CTAs for the machine, at least 16 columns, clusters of up to 8
  const bool v4 = sh.vdim % 4 == 0 && ((uintptr_t)a.state % 16) == 0;
  const int V = v4 ? 4 : 1;
  int ranks = 1;
  while (ranks < 8 && (int64_t)a.B * sh.H * ranks < 2 * st->sm_count && sh.vdim / (2 * ranks) >= 16) ranks *= 2;
  auto cols = [&](int r) { return ((sh.vdim + r - 1) / r + V - 1) / V * V; };
  while (cols(ranks) / V > kMsThreads && ranks < 8) ranks *= 2;
  while (ranks > 1 && (int64_t)(ranks - 1) * cols(ranks) >= sh.vdim) ranks /= 2;   // every rank has columns
  const int cw = cols(ranks);
  TSB_CHECK(cw / V <= kMsThreads, "matrix memory: values of %d elements are not supported", sh.vdim);
  const size_t smem = ((size_t)3 * sh.dim + cw + (size_t)(kMsThreads / (cw / V)) * cw + 32) * sizeof(float);
  TSB_CHECK(smem <= 160 * 1024, "matrix memory: keys of %d elements are not supported", sh.dim);
  if (dtype == TSB200_F32) return v4 ? memory_step_go<float, 4>(device, a, ranks, cw, smem, s) : memory_step_go<float, 1>(device, a, ranks, cw, smem, s);
  return v4 ? memory_step_go<bf16, 4>(device, a, ranks, cw, smem, s) : memory_step_go<bf16, 1>(device, a, ranks, cw, smem, s);
}

}  // namespace tsb
