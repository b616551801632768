// Latent attention: the cache keeps one vector per position, [latent c (rank) | rotated key part shared by all heads (rot)], and every
// head's keys and values are linear images of c.  score = (q_n . (Uk_h c) + q_r . k_r) * scale, value = Uv_h c.
//
// Two forms of the same product:
//   absorbed   q_lat = [Uk_h^T q_n | q_r] once per query, then all heads attend to the cache rows themselves (one key of
//              rank + rot elements whose first rank elements are also the value), and Uv_h is applied to the result.  Reads the cache
//              once for all heads: decoding and short portions.
//                latent_query_kernel     q_lat (Uk read once per eight rows, its inner dimension split over the warps)
//                latent_attn_mma_kernel  bf16, split over the key range: 16 (query, head) rows per CTA on mma.sync, cache rows
//                                        staged once by cp.async as keys AND values; scores meet in shared memory so that each
//                                        warp can own a slice of the latent in the second product
//                latent_attn_kernel      any type and size up to a latent of 1024, CUDA cores
//                latent_value_kernel     merges the splits and applies Uv_h
//   expanded   keys and values of all heads are materialised from the cache rows by one tensor-core linear, then causal flash
//              attention per head (latent_prefill_mma_kernel: 128 queries per CTA, mma.sync).  Fewer operations per (query, key)
//              pair, paid for by the expansion: long portions.
// Scores, softmax and sums are fp32 in every kernel; positions and angles come from a table computed in double precision.
#include "kernels.cuh"

namespace tsb {

TSB_CHECKED_WORD(latent)
#ifndef TSB200_CHECKED
int chk_take_latent() { return 0; }
#endif

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ void la_ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void la_ldsm_x2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void la_ldsm_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
// 16 bytes to shared memory; with live == false the destination is zero-filled and the source is not read
__device__ __forceinline__ void la_cp16(uint32_t dst, const void* src, bool live = true) {
  const int n = live ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void la_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void la_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ uint32_t la_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

__global__ void angle_table_kernel(float2* tab, int Tmax, int dims, double base) {
  const int half = dims / 2;
  const int64_t n = (int64_t)Tmax * half;
  for (int64_t p = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; p < n; p += (int64_t)gridDim.x * blockDim.x) {
    const double a = (double)(p / half) * pow(base, -2.0 * (double)(p % half) / (double)dims);
    tab[p] = make_float2((float)cos(a), (float)sin(a));
  }
}

// (u, v) at (i, i + dims / 2) of the first `dims` values of `p`
template <typename T>
__device__ __forceinline__ void turn_pair(const T* src, T* dst, int i, int dims, const float2 cs) {
  const float u = to_f<T>(src[i]), v = to_f<T>(src[i + dims / 2]);
  dst[i] = from_f<T>(u * cs.x - v * cs.y);
  dst[i + dims / 2] = from_f<T>(v * cs.x + u * cs.y);
}

constexpr int kLatentAppendThreads = 128;
template <typename T>
__global__ void __launch_bounds__(kLatentAppendThreads) latent_append_kernel(LatentShape a, T* qkv, int row_stride, int dkv_col, const T* norm_w, float eps,
                                                                             T* cache, int64_t seq_stride, int S, int T0_arg, const int* state, int Tmax,
                                                                             const float2* tab) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x, b = row / S, tid = threadIdx.x;
  const int pos = state_len(state, b, T0_arg) + row % S;
  TSB_DEV_CHECK(latent, pos >= 0 && pos < Tmax, 0x601, return)   // append position outside the cache
  if (pos >= Tmax) return;   // capacity is checked on the host; never write past the cache
  const int half = a.rot_dims / 2;
  const float2* cs = tab + (int64_t)pos * half;
  T* q = qkv + (int64_t)row * row_stride;
  for (int p = tid; p < a.H * half; p += kLatentAppendThreads) {
    T* r = q + (int64_t)(p / half) * (a.dim + a.rot) + a.dim;
    turn_pair<T>(r, r, p % half, a.rot_dims, cs[p % half]);
  }
  if (dkv_col < 0) return;
  const T* x = q + dkv_col;
  T* out = cache + (int64_t)b * seq_stride + (int64_t)pos * a.row;
  float s = 0.0f;
  for (int i = tid; i < a.rank; i += kLatentAppendThreads) {
    const float v = to_f<T>(x[i]);
    s += v * v;
  }
  s = block_sum(s, red);
  const float inv = 1.0f / sqrtf(s / (float)a.rank + eps);
  for (int i = tid; i < a.rank; i += kLatentAppendThreads) out[i] = from_f<T>(to_f<T>(x[i]) * inv * to_f<T>(norm_w[i]));
  for (int i = tid; i < half; i += kLatentAppendThreads) turn_pair<T>(x + a.rank, out + a.rank, i, a.rot_dims, cs[i]);
  for (int i = a.rot_dims + tid; i < a.rot; i += kLatentAppendThreads) out[a.rank + i] = x[a.rank + i];
}

// q_lat[row, h, :] = [sum_d q[row, h, d] Uk[h * dim + d, :] | rotated part | zeros]
constexpr int kLqThreads = 256, kLqCols = 64, kLqRows = 8;
template <typename T>
__global__ void __launch_bounds__(kLqThreads) latent_query_kernel(LatentShape a, T* q_lat, const T* q, int q_stride, const T* uk, int rows) {
  extern __shared__ float s_q[];              // [8 rows][dim]
  __shared__ float s_red[8][kLqRows][kLqCols];
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, c0 = blockIdx.y * kLqCols, r0 = blockIdx.z * kLqRows;
  const int n = min(kLqRows, rows - r0);
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
  for (int i = tid; i < kLqRows * a.dim; i += kLqThreads) {
    const int r = i / a.dim;
    s_q[i] = r < n ? to_f<T>(q[(int64_t)(r0 + r) * q_stride + (int64_t)h * (a.dim + a.rot) + i % a.dim]) : 0.0f;
  }
  if (blockIdx.y == 0) {
    const int tail = a.row - a.rank;
    for (int i = tid; i < n * tail; i += kLqThreads) {
      const int r = i / tail, e = i % tail;
      const T v = e < a.rot ? q[(int64_t)(r0 + r) * q_stride + (int64_t)h * (a.dim + a.rot) + a.dim + e] : from_f<T>(0.0f);
      q_lat[((int64_t)(r0 + r) * a.H + h) * a.row + a.rank + e] = v;
    }
  }
  __syncthreads();
  const int c = c0 + lane * 2;
  float acc[kLqRows][2];
#pragma unroll
  for (int r = 0; r < kLqRows; ++r) acc[r][0] = acc[r][1] = 0.0f;
  const bool in0 = c < a.rank, in1 = c + 1 < a.rank;
#pragma unroll 8
  for (int dd = w; dd < a.dim; dd += 8) {
    const T* u = uk + ((int64_t)h * a.dim + dd) * a.rank + c;
    const float u0 = in0 ? to_f<T>(u[0]) : 0.0f, u1 = in1 ? to_f<T>(u[1]) : 0.0f;
#pragma unroll
    for (int r = 0; r < kLqRows; ++r) {
      acc[r][0] = fmaf(s_q[r * a.dim + dd], u0, acc[r][0]);
      acc[r][1] = fmaf(s_q[r * a.dim + dd], u1, acc[r][1]);
    }
  }
#pragma unroll
  for (int r = 0; r < kLqRows; ++r) {
    s_red[w][r][lane * 2] = acc[r][0];
    s_red[w][r][lane * 2 + 1] = acc[r][1];
  }
  __syncthreads();
  for (int i = tid; i < n * kLqCols; i += kLqThreads) {
    const int r = i / kLqCols, e = i % kLqCols;
    if (c0 + e >= a.rank) continue;
    float v = 0.0f;
#pragma unroll
    for (int q8 = 0; q8 < 8; ++q8) v += s_red[q8][r][e];
    q_lat[((int64_t)(r0 + r) * a.H + h) * a.row + c0 + e] = from_f<T>(v);
  }
}

// ---- absorbed form on CUDA cores: one CTA per (query, head) row and split -------------------------------------------------------
template <typename T, int NI>   // NI * 32 >= latent size
__global__ void __launch_bounds__(256) latent_attn_kernel(LatentShape a, float* part, const T* q_lat, const T* cache, int64_t seq_stride, int S, int T0_arg,
                                                          const int* state, int Tmax, int splits) {
  extern __shared__ float sm[];   // the query row [row], then the warps' states [8][rank + 2]
  pdl_trigger();
  pdl_wait();
  const int64_t rr = blockIdx.x;   // (b * S + s) * H + h
  const int row = (int)(rr / a.H), b = row / S, s = row % S, split = blockIdx.y;
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
  const int n_keys = min(state_len(state, b, T0_arg) + s + 1, Tmax);
  const int per = (n_keys + splits - 1) / splits;
  const int t0 = split * per, t1 = min(n_keys, t0 + per);
  for (int i = tid; i < a.row; i += 256) sm[i] = to_f<T>(q_lat[rr * a.row + i]) * a.scale;
  __syncthreads();
  float m = -INFINITY, l = 0.0f, o[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) o[i] = 0.0f;
  for (int t = t0 + w; t < t1; t += 8) {
    const T* k = cache + (int64_t)b * seq_stride + (int64_t)t * a.row;
    float kv[NI], z = 0.0f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int e = lane + 32 * i;
      kv[i] = e < a.rank ? to_f<T>(k[e]) : 0.0f;
      z = fmaf(kv[i], e < a.rank ? sm[e] : 0.0f, z);
    }
    for (int e = a.rank + lane; e < a.rank + a.rot; e += 32) z = fmaf(to_f<T>(k[e]), sm[e], z);
    z = warp_sum(z);
    const float mn = fmaxf(m, z), corr = expf(m - mn), p = expf(z - mn);
    l = l * corr + p;
    m = mn;
#pragma unroll
    for (int i = 0; i < NI; ++i) o[i] = o[i] * corr + p * kv[i];
  }
  const int rec = a.rank + 2;
  float* st = sm + a.row;
  if (lane == 0) {
    st[w * rec] = m;
    st[w * rec + 1] = l;
  }
#pragma unroll
  for (int i = 0; i < NI; ++i)
    if (lane + 32 * i < a.rank) st[w * rec + 2 + lane + 32 * i] = o[i];
  __syncthreads();
  float mx = -INFINITY;
  for (int q = 0; q < 8; ++q) mx = fmaxf(mx, st[q * rec]);
  float* out = part + (rr * splits + split) * rec;
  for (int e = tid; e < a.rank + 1; e += 256) {
    float v = 0.0f;
    for (int q = 0; q < 8; ++q) v += (st[q * rec] == -INFINITY) ? 0.0f : st[q * rec + 1 + e] * expf(st[q * rec] - mx);
    out[1 + e] = v;
  }
  if (tid == 0) out[0] = mx;
}

// ---- absorbed form on the warp-level tensor cores -------------------------------------------------------------------------------
constexpr int kLmThreads = 256, kLmKeys = 64;
struct LatentMmaLayout {   // shared memory of latent_attn_mma_kernel
  int pitch;               // bytes of a staged row: an odd number of 16-byte units, so that ldmatrix rows fall into different banks
  int stages;
  size_t stage_bytes, q_off, s_off, p_off, st_off, total;
};
__host__ __device__ inline LatentMmaLayout latent_mma_layout(int row, int stages) {
  LatentMmaLayout L;
  L.pitch = row * 2 + 16;
  L.stages = stages;
  L.stage_bytes = (size_t)kLmKeys * L.pitch;
  L.q_off = L.stage_bytes * stages;
  L.s_off = L.q_off + (size_t)16 * L.pitch;
  L.p_off = L.s_off + 16 * (kLmKeys + 4) * 4;
  L.st_off = L.p_off + 16 * (kLmKeys + 8) * 2;
  L.total = L.st_off + 48 * 4;
  return L;
}

template <int NBW>   // latent blocks of 8 columns a warp owns in the second product (even)
__global__ void __launch_bounds__(kLmThreads) latent_attn_mma_kernel(LatentShape a, float* part, const bf16* q_lat, const bf16* cache, int64_t seq_stride,
                                                                     int S, int T0_arg, const int* state, int Tmax, int splits, int stages) {
  extern __shared__ __align__(128) unsigned char smem[];
  pdl_trigger();
  pdl_wait();
  const LatentMmaLayout L = latent_mma_layout(a.row, stages);
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
  const int split = blockIdx.x, r0 = blockIdx.y * 16, b = blockIdx.z;
  const int R = S * a.H;                       // (query, head) rows of the sequence
  const int T0 = state_len(state, b, T0_arg);
  const int s_last = (min(r0 + 16, R) - 1) / a.H;
  const int n_keys = min(T0 + s_last + 1, Tmax);
  const int per = (n_keys + splits - 1) / splits;
  const int t_beg = split * per, t_end = min(n_keys, t_beg + per);
  const int n_tiles = (max(t_end - t_beg, 0) + kLmKeys - 1) / kLmKeys;
  const bf16* base = cache + (int64_t)b * seq_stride;
  const int cpr = a.row / 8;                   // 16-byte chunks per row
  const uint32_t sbase = la_smem(smem);
  float* sS = reinterpret_cast<float*>(smem + L.s_off);
  bf16* sP = reinterpret_cast<bf16*>(smem + L.p_off);
  float* s_m = reinterpret_cast<float*>(smem + L.st_off);
  float *s_l = s_m + 16, *s_c = s_m + 32;
  constexpr int SP = kLmKeys + 4, PP = kLmKeys + 8;

  auto issue = [&](int tile) {
    if (tile < n_tiles) {
      const uint32_t dst = sbase + (uint32_t)((tile % stages) * L.stage_bytes);
      const int t0 = t_beg + tile * kLmKeys;
      for (int v = tid; v < kLmKeys * cpr; v += kLmThreads) {
        const int tt = v / cpr, c = v % cpr;
        const int t = min(t0 + tt, t_end - 1);   // the tail re-reads the last key of the range; its scores are masked
        la_cp16(dst + tt * L.pitch + c * 16, base + (int64_t)t * a.row + c * 8);
      }
    }
    la_commit();
  };
  issue(0);
  {
    const bf16* src = q_lat + ((int64_t)b * R + r0) * a.row;
    for (int v = tid; v < 16 * cpr; v += kLmThreads) {
      const int rr = v / cpr, c = v % cpr;
      uint4 x = make_uint4(0, 0, 0, 0);
      if (r0 + rr < R) x = *reinterpret_cast<const uint4*>(src + (int64_t)rr * a.row + c * 8);
      *reinterpret_cast<uint4*>(smem + L.q_off + rr * L.pitch + c * 16) = x;
    }
    if (tid < 16) {
      s_m[tid] = -INFINITY;
      s_l[tid] = 0.0f;
    }
  }
  float o[NBW][4];
#pragma unroll
  for (int i = 0; i < NBW; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
  const int col0 = w * NBW * 8;                // first latent column of this warp
  const int ksteps = a.row / 16;
  // softmax: thread -> row tid / 16, four keys from (tid % 16) * 4
  const int sr = tid >> 4, sc0 = (tid & 15) * 4;
  const int row_lim = r0 + sr < R ? T0 + (r0 + sr) / a.H + 1 : 0;   // keys [0, row_lim) are visible

  for (int tile = 0; tile < n_tiles; ++tile) {
    if (stages > 1) {
      issue(tile + 1);
      la_wait<1>();
    } else {
      if (tile > 0) issue(tile);
      la_wait<0>();
    }
    __syncthreads();
    const uint32_t kb = sbase + (uint32_t)((tile % stages) * L.stage_bytes);
    {   // scores of keys w * 8 .. + 7
      float c0[4] = {0.0f, 0.0f, 0.0f, 0.0f}, c1[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      const uint32_t qa = sbase + (uint32_t)L.q_off + (lane & 15) * L.pitch + (lane >> 4) * 16;
      const uint32_t ka = kb + (w * 8 + (lane & 7)) * L.pitch + (lane >> 3) * 16;
      int ks = 0;
#pragma unroll 2
      for (; ks + 1 < ksteps; ks += 2) {
        uint32_t a0, a1, a2, a3, b0, b1, b2, b3;
        la_ldsm_x4(ka + ks * 32, b0, b1, b2, b3);
        la_ldsm_x4(qa + ks * 32, a0, a1, a2, a3);
        mma_16816<bf16>(c0, a0, a1, a2, a3, b0, b1);
        la_ldsm_x4(qa + ks * 32 + 32, a0, a1, a2, a3);
        mma_16816<bf16>(c1, a0, a1, a2, a3, b2, b3);
      }
      if (ks < ksteps) {
        uint32_t a0, a1, a2, a3, b0, b1;
        la_ldsm_x2(kb + (w * 8 + (lane & 7)) * L.pitch + ((lane >> 3) & 1) * 16 + ks * 32, b0, b1);
        la_ldsm_x4(qa + ks * 32, a0, a1, a2, a3);
        mma_16816<bf16>(c0, a0, a1, a2, a3, b0, b1);
      }
      float* d = sS + w * 8 + 2 * t4;
      *reinterpret_cast<float2*>(d + g8 * SP) = make_float2(c0[0] + c1[0], c0[1] + c1[1]);
      *reinterpret_cast<float2*>(d + (g8 + 8) * SP) = make_float2(c0[2] + c1[2], c0[3] + c1[3]);
    }
    __syncthreads();
    {
      const int t0 = t_beg + tile * kLmKeys + sc0;
      const float4 z4 = *reinterpret_cast<const float4*>(sS + sr * SP + sc0);
      float z[4] = {z4.x, z4.y, z4.z, z4.w};
      float mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        z[e] = (t0 + e < t_end && t0 + e < row_lim) ? z[e] * a.scale : -INFINITY;
        mx = fmaxf(mx, z[e]);
      }
#pragma unroll
      for (int q = 8; q > 0; q >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, q));
      const float m_old = s_m[sr], m_new = fmaxf(m_old, mx);
      float p[4], sum = 0.0f;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        p[e] = m_new == -INFINITY ? 0.0f : __expf(z[e] - m_new);   // a row may see none of these keys
        sum += p[e];
      }
#pragma unroll
      for (int q = 8; q > 0; q >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, q);
      *reinterpret_cast<uint2*>(sP + sr * PP + sc0) = make_uint2(Pair16<bf16>::put(p[0], p[1]), Pair16<bf16>::put(p[2], p[3]));
      if ((tid & 15) == 0) {
        const float corr = m_new == -INFINITY ? 1.0f : __expf(m_old - m_new);
        s_c[sr] = corr;
        s_m[sr] = m_new;
        s_l[sr] = s_l[sr] * corr + sum;
      }
    }
    __syncthreads();
    {
      const float cA = s_c[g8], cB = s_c[g8 + 8];
#pragma unroll
      for (int i = 0; i < NBW; ++i) {
        o[i][0] *= cA; o[i][1] *= cA; o[i][2] *= cB; o[i][3] *= cB;
      }
      const uint32_t pa = la_smem(sP) + (lane & 15) * (PP * 2) + (lane >> 4) * 16;
      const uint32_t va = kb + ((lane & 7) + ((lane >> 3) & 1) * 8) * L.pitch + (lane >> 4) * 16;
#pragma unroll
      for (int ks = 0; ks < kLmKeys / 16; ++ks) {
        uint32_t a0, a1, a2, a3;
        la_ldsm_x4(pa + ks * 32, a0, a1, a2, a3);
#pragma unroll
        for (int i = 0; i < NBW; i += 2) {
          const int col = col0 + i * 8;
          if (col < a.row) {   // the row is a multiple of 16 elements: both blocks of the pair are inside
            uint32_t b0, b1, b2, b3;
            la_ldsm_x4_trans(va + ks * 16 * L.pitch + col * 2, b0, b1, b2, b3);
            mma_16816<bf16>(o[i], a0, a1, a2, a3, b0, b1);
            mma_16816<bf16>(o[i + 1], a0, a1, a2, a3, b2, b3);
          }
        }
      }
    }
    __syncthreads();   // the stage is overwritten by the copy issued in the next iteration
  }
  la_wait<0>();
  const int rec = a.rank + 2;
  float* pb = part + (((int64_t)b * R + r0) * splits + split) * rec;
  if (n_tiles == 0) __syncthreads();   // the initial states of an empty range
#pragma unroll
  for (int i = 0; i < NBW; ++i) {
    const int col = col0 + i * 8 + 2 * t4;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int rr = g8 + (e >> 1) * 8, c = col + (e & 1);
      if (r0 + rr < R && c < a.rank) pb[(int64_t)rr * splits * rec + 2 + c] = o[i][e];
    }
  }
  if (tid < 16 && r0 + tid < R) {
    pb[(int64_t)tid * splits * rec] = s_m[tid];
    pb[(int64_t)tid * splits * rec + 1] = s_l[tid];
  }
}

// merges the splits of a (query, head) row and applies Uv_h: 32 value elements per CTA
constexpr int kLvThreads = 256, kLvCols = 32;
template <typename T>
__global__ void __launch_bounds__(kLvThreads) latent_value_kernel(LatentShape a, T* out, const float* part, const T* uv, int splits) {
  extern __shared__ float s_o[];
  pdl_trigger();
  pdl_wait();
  const int64_t rr = blockIdx.x;
  const int h = (int)(rr % a.H), v0 = blockIdx.y * kLvCols;
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, rec = a.rank + 2;
  const float* p = part + rr * splits * rec;
  float mx = -INFINITY, l = 0.0f;
  for (int i = 0; i < splits; ++i) mx = fmaxf(mx, p[(int64_t)i * rec]);
  for (int i = 0; i < splits; ++i) {
    const float m = p[(int64_t)i * rec];
    l += m == -INFINITY ? 0.0f : p[(int64_t)i * rec + 1] * expf(m - mx);
  }
  const float inv = l > 0.0f ? 1.0f / l : 0.0f;
  for (int e = tid; e < a.rank; e += kLvThreads) {
    float v = 0.0f;
    for (int i = 0; i < splits; ++i) {
      const float m = p[(int64_t)i * rec];
      v += m == -INFINITY ? 0.0f : p[(int64_t)i * rec + 2 + e] * expf(m - mx);
    }
    s_o[e] = v * inv;
  }
  __syncthreads();
  for (int q = w; q < kLvCols && v0 + q < a.vdim; q += 8) {
    const T* u = uv + ((int64_t)h * a.vdim + v0 + q) * a.rank;
    float acc = 0.0f;
    if constexpr (sizeof(T) == 2) {
      if (a.rank % 2 == 0) {
#pragma unroll 4
        for (int e = lane * 2; e < a.rank; e += 64) {
          const float2 t = Pair16<bf16>::get(*reinterpret_cast<const uint32_t*>(u + e));
          acc = fmaf(t.x, s_o[e], acc);
          acc = fmaf(t.y, s_o[e + 1], acc);
        }
      } else {
        for (int e = lane; e < a.rank; e += 32) acc = fmaf(to_f<T>(u[e]), s_o[e], acc);
      }
    } else {
      for (int e = lane; e < a.rank; e += 32) acc = fmaf(to_f<T>(u[e]), s_o[e], acc);
    }
    acc = warp_sum(acc);
    if (lane == 0) out[rr * a.vdim + v0 + q] = from_f<T>(acc);
  }
}

// ---- expanded form: causal flash attention over materialised keys and values ----------------------------------------------------
constexpr int kLpThreads = 256, kLpRows = 128, kLpKeys = 64;
template <int VN>   // value blocks of 8 columns (vdim <= VN * 8)
__global__ void __launch_bounds__(kLpThreads, VN <= 16 ? 2 : 1) latent_prefill_mma_kernel(LatentShape a, bf16* out, const bf16* q, int q_stride, const bf16* kv,
                                                                                         const bf16* cache, int64_t seq_stride, int S, int T0, int qk) {
  extern __shared__ __align__(128) unsigned char smem[];
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
  const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kLpRows, h = blockIdx.y, b = blockIdx.z;   // the longest key ranges start first
  const int qpitch = qk * 2 + 16, vpitch = VN * 16 + 16;
  const uint32_t sq = la_smem(smem), sk = sq + kLpRows * qpitch;
  const uint32_t stage = kLpKeys * (qpitch + vpitch);
  const int kvw = a.H * (a.dim + a.vdim);
  const bf16* kvb = kv + (int64_t)b * (T0 + S) * kvw;
  const bf16* cb = cache + (int64_t)b * seq_stride;
  const int n_keys = T0 + min(S, q0 + kLpRows);
  const int w_keys = min(T0 + q0 + w * 16 + 16, n_keys);
  const int n_tiles = (n_keys + kLpKeys - 1) / kLpKeys;
  const int qc = qk / 8, dc = a.dim / 8, rc = a.rot / 8, vc = a.vdim / 8;

  auto issue = [&](int tile) {
    if (tile < n_tiles) {
      const uint32_t dk = sk + (uint32_t)(tile & 1) * stage, dv = dk + kLpKeys * qpitch;
      const int t0 = tile * kLpKeys;
      for (int v = tid; v < kLpKeys * qc; v += kLpThreads) {
        const int tt = v / qc, c = v % qc, t = min(t0 + tt, n_keys - 1);
        const bf16* src = c < dc ? kvb + (int64_t)t * kvw + h * a.dim + c * 8 : cb + (int64_t)t * a.row + a.rank + (c < dc + rc ? c - dc : 0) * 8;
        la_cp16(dk + tt * qpitch + c * 16, src, c < dc + rc);
      }
      for (int v = tid; v < kLpKeys * VN; v += kLpThreads) {
        const int tt = v / VN, c = v % VN, t = min(t0 + tt, n_keys - 1);
        la_cp16(dv + tt * vpitch + c * 16, kvb + (int64_t)t * kvw + a.H * a.dim + h * a.vdim + (c < vc ? c : 0) * 8, c < vc);
      }
    }
    la_commit();
  };
  {
    const int per = a.dim + a.rot;
    for (int v = tid; v < kLpRows * qc; v += kLpThreads) {
      const int rr = v / qc, c = v % qc, s = q0 + rr;
      const bool live = s < S && c < dc + rc;
      la_cp16(sq + rr * qpitch + c * 16, q + ((int64_t)b * S + (live ? s : 0)) * q_stride + h * per + (live ? c : 0) * 8, live);
    }
  }
  issue(0);
  const int sA = q0 + w * 16 + g8, sB = sA + 8;
  const int limA = sA < S ? T0 + sA + 1 : 0, limB = sB < S ? T0 + sB + 1 : 0;
  float mA = -INFINITY, mB = -INFINITY, lA = 0.0f, lB = 0.0f;
  float o[VN][4];
#pragma unroll
  for (int i = 0; i < VN; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
  const uint32_t qa = sq + (w * 16 + (lane & 15)) * qpitch + (lane >> 4) * 16;
  const int ksteps = qk / 16;

  for (int tile = 0; tile < n_tiles; ++tile) {
    issue(tile + 1);
    la_wait<1>();
    __syncthreads();
    const uint32_t kb = sk + (uint32_t)(tile & 1) * stage, vb = kb + kLpKeys * qpitch;
#pragma unroll 1
    for (int sl = 0; sl < kLpKeys / 32; ++sl) {
      const int t_first = tile * kLpKeys + sl * 32;
      if (t_first >= w_keys) break;   // causal: nothing further in this stage is visible to this warp (warp-uniform)
      float sc[4][4];
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[nb][e] = 0.0f;
      // K fragments of two 8-key blocks per ldmatrix: lanes 0-7 / 8-15 keys 0-7, k chunks 0 / 1; lanes 16-31 keys 8-15
      const uint32_t ka = kb + (sl * 32 + (lane & 7) + ((lane >> 4) << 3)) * qpitch + ((lane >> 3) & 1) * 16;
#pragma unroll 2
      for (int ks = 0; ks < ksteps; ++ks) {
        uint32_t a0, a1, a2, a3, b0, b1, b2, b3;
        la_ldsm_x4(qa + ks * 32, a0, a1, a2, a3);
        la_ldsm_x4(ka + ks * 32, b0, b1, b2, b3);
        mma_16816<bf16>(sc[0], a0, a1, a2, a3, b0, b1);
        mma_16816<bf16>(sc[1], a0, a1, a2, a3, b2, b3);
        la_ldsm_x4(ka + 16 * qpitch + ks * 32, b0, b1, b2, b3);
        mma_16816<bf16>(sc[2], a0, a1, a2, a3, b0, b1);
        mma_16816<bf16>(sc[3], a0, a1, a2, a3, b2, b3);
      }
      float mxA = -INFINITY, mxB = -INFINITY;
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = t_first + nb * 8 + 2 * t4 + e;
          sc[nb][e] = t < limA ? sc[nb][e] * a.scale : -INFINITY;
          sc[nb][2 + e] = t < limB ? sc[nb][2 + e] * a.scale : -INFINITY;
          mxA = fmaxf(mxA, sc[nb][e]);
          mxB = fmaxf(mxB, sc[nb][2 + e]);
        }
      mxA = fmaxf(mxA, __shfl_xor_sync(0xffffffffu, mxA, 1));
      mxA = fmaxf(mxA, __shfl_xor_sync(0xffffffffu, mxA, 2));
      mxB = fmaxf(mxB, __shfl_xor_sync(0xffffffffu, mxB, 1));
      mxB = fmaxf(mxB, __shfl_xor_sync(0xffffffffu, mxB, 2));
      const float nA = fmaxf(mA, mxA), nB = fmaxf(mB, mxB);
      const float cA = nA == -INFINITY ? 1.0f : __expf(mA - nA), cB = nB == -INFINITY ? 1.0f : __expf(mB - nB);
      float suA = 0.0f, suB = 0.0f;
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          sc[nb][e] = nA == -INFINITY ? 0.0f : __expf(sc[nb][e] - nA);
          sc[nb][2 + e] = nB == -INFINITY ? 0.0f : __expf(sc[nb][2 + e] - nB);
          suA += sc[nb][e];
          suB += sc[nb][2 + e];
        }
      lA = lA * cA + suA;
      lB = lB * cB + suB;
      mA = nA;
      mB = nB;
#pragma unroll
      for (int i = 0; i < VN; ++i) {
        o[i][0] *= cA; o[i][1] *= cA; o[i][2] *= cB; o[i][3] *= cB;
      }
#pragma unroll
      for (int kk = 0; kk < 2; ++kk) {
        const uint32_t p0 = Pair16<bf16>::put(sc[2 * kk][0], sc[2 * kk][1]), p1 = Pair16<bf16>::put(sc[2 * kk][2], sc[2 * kk][3]);
        const uint32_t p2 = Pair16<bf16>::put(sc[2 * kk + 1][0], sc[2 * kk + 1][1]), p3 = Pair16<bf16>::put(sc[2 * kk + 1][2], sc[2 * kk + 1][3]);
        const uint32_t va = vb + (sl * 32 + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vpitch + (lane >> 4) * 16;
#pragma unroll
        for (int i = 0; i < VN; i += 2) {
          uint32_t b0, b1, b2, b3;
          la_ldsm_x4_trans(va + i * 16, b0, b1, b2, b3);
          mma_16816<bf16>(o[i], p0, p1, p2, p3, b0, b1);
          mma_16816<bf16>(o[i + 1], p0, p1, p2, p3, b2, b3);
        }
      }
    }
    __syncthreads();
  }
  la_wait<0>();
  lA += __shfl_xor_sync(0xffffffffu, lA, 1);
  lA += __shfl_xor_sync(0xffffffffu, lA, 2);
  lB += __shfl_xor_sync(0xffffffffu, lB, 1);
  lB += __shfl_xor_sync(0xffffffffu, lB, 2);
  const float iA = lA > 0.0f ? 1.0f / lA : 0.0f, iB = lB > 0.0f ? 1.0f / lB : 0.0f;
#pragma unroll
  for (int i = 0; i < VN; ++i) {
    const int c = i * 8 + 2 * t4;
    if (c >= a.vdim) continue;   // vdim is a multiple of 8
    if (sA < S) *reinterpret_cast<uint32_t*>(out + (((int64_t)b * S + sA) * a.H + h) * a.vdim + c) = Pair16<bf16>::put(o[i][0] * iA, o[i][1] * iA);
    if (sB < S) *reinterpret_cast<uint32_t*>(out + (((int64_t)b * S + sB) * a.H + h) * a.vdim + c) = Pair16<bf16>::put(o[i][2] * iB, o[i][3] * iB);
  }
}

// ---- host side ------------------------------------------------------------------------------------------------------------------
int launch_angle_table(int device, DeviceState* st, float2* tab, int Tmax, int dims, double base, cudaStream_t s) {
  const int64_t n = (int64_t)Tmax * (dims / 2);
  int64_t g = (n + 255) / 256;
  if (g > (int64_t)st->sm_count * 8) g = (int64_t)st->sm_count * 8;
  angle_table_kernel<<<(int)(g > 0 ? g : 1), 256, 0, s>>>(tab, Tmax, dims, base);
  count_launch(device);
  return check_launch("angle_table");
}

int launch_latent_append(int device, int dtype, const LatentShape& a, void* qkv, int row_stride, int dkv_col, const void* norm_w, float eps, void* cache,
                         int64_t seq_stride, int B, int S, int T0, const int* state, int Tmax, const float2* tab, cudaStream_t s) {
  TSB_CHECK(state || T0 + S <= Tmax, "latent_append: cache capacity exceeded (%d + %d > %d)", T0, S, Tmax);
  if (dtype == TSB200_F32)
    TSB_CUDA(launch_k(latent_append_kernel<float>, dim3(B * S), dim3(kLatentAppendThreads), 0, s, a, (float*)qkv, row_stride, dkv_col, (const float*)norm_w,
                      eps, (float*)cache, seq_stride, S, T0, state, Tmax, tab));
  else
    TSB_CUDA(launch_k(latent_append_kernel<bf16>, dim3(B * S), dim3(kLatentAppendThreads), 0, s, a, (bf16*)qkv, row_stride, dkv_col, (const bf16*)norm_w, eps,
                      (bf16*)cache, seq_stride, S, T0, state, Tmax, tab));
  count_launch(device);
  return check_launch("latent_append");
}

constexpr size_t kLatentSmemMax = 226 * 1024;
static bool latent_mma_shape(int dtype, const LatentShape& a) {
  return dtype == TSB200_BF16 && a.rank % 8 == 0 && a.rank <= 1024 && latent_mma_layout(a.row, 1).total <= kLatentSmemMax;
}

// splits of the key range: about one CTA per SM, at least 64 keys each
int latent_pick_splits(DeviceState* st, const LatentShape& a, int B, int S, int T) {
  const int64_t base = (int64_t)B * (((int64_t)S * a.H + 15) / 16);
  int64_t n = (st->sm_count + base / 2) / base;
  const int by_len = (T + 63) / 64;
  if (n > by_len) n = by_len;
  if (n > 64) n = 64;
  return n < 1 ? 1 : (int)n;
}

static size_t latent_prefill_smem(int qk, int vn) { return (size_t)kLpRows * (qk * 2 + 16) + 2 * (size_t)kLpKeys * (qk * 2 + 16 + vn * 16 + 16); }
static int latent_vn(int vdim) { return vdim <= 32 ? 4 : (vdim <= 64 ? 8 : (vdim <= 128 ? 16 : 32)); }

// The expanded form: per (query, key) pair and head dim + rot + vdim products instead of 2 rank + rot, plus rank (dim + vdim) per key
// shared by the S queries of the portion.
bool latent_expanded(int dtype, const LatentShape& a, int q_stride, int S) {
  if (dtype != TSB200_BF16 || S < 16) return false;
  if (a.dim % 8 || a.rot % 8 || a.vdim % 8 || a.rank % 8 || q_stride % 8 || a.vdim > 256) return false;
  const int qk = (a.dim + a.rot + 15) / 16 * 16;
  if (latent_prefill_smem(qk, latent_vn(a.vdim)) > kLatentSmemMax) return false;
  const double expanded = (double)(a.dim + a.rot + a.vdim) + (double)a.rank * (a.dim + a.vdim) / S;
  return expanded < (double)(2 * a.rank + a.rot);
}

template <typename T>
static int latent_simple(int device, const LatentArgs& a, cudaStream_t s) {
  const LatentShape& sh = a.shape;
  const size_t smem = ((size_t)sh.row + 8 * (sh.rank + 2)) * sizeof(float);
  const dim3 grid(a.B * a.S * sh.H, a.splits);
  static bool done[kMaxDevices] = {};
  if (!done[device]) {
    TSB_CUDA(cudaFuncSetAttribute(latent_attn_kernel<T, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024));
    TSB_CUDA(cudaFuncSetAttribute(latent_attn_kernel<T, 16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024));
    TSB_CUDA(cudaFuncSetAttribute(latent_attn_kernel<T, 32>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024));
    done[device] = true;
  }
  TSB_CHECK(sh.rank <= 1024 && smem <= 64 * 1024, "latent attention: a latent of %d is not supported (at most 1024)", sh.rank);
  auto k = sh.rank <= 128 ? latent_attn_kernel<T, 4> : (sh.rank <= 512 ? latent_attn_kernel<T, 16> : latent_attn_kernel<T, 32>);
  TSB_CUDA(launch_k(k, grid, dim3(256), smem, s, sh, a.part, (const T*)a.q_lat, (const T*)a.cache, a.seq_stride, a.S, a.T0, a.state, a.Tmax, a.splits));
  return 1;
}

template <typename T>
static int latent_absorbed(int device, int dtype, const LatentArgs& a, cudaStream_t s) {
  const LatentShape& sh = a.shape;
  const int rows = a.B * a.S;
  TSB_CHECK((int64_t)rows * sh.H * a.splits * (sh.rank + 2) <= a.part_elems, "latent attention: scratch too small for %d rows in %d splits", rows, a.splits);
  const size_t sq = (size_t)kLqRows * sh.dim * sizeof(float);
  TSB_CHECK(sq <= 24 * 1024, "latent attention: unrotated head size %d is not supported (at most 768)", sh.dim);
  TSB_CUDA(launch_k(latent_query_kernel<T>, dim3(sh.H, (sh.rank + kLqCols - 1) / kLqCols, (rows + kLqRows - 1) / kLqRows), dim3(kLqThreads), sq, s, sh,
                    (T*)a.q_lat, (const T*)a.q, a.q_stride, (const T*)a.uk, rows));
  count_launch(device);
  bool done_mma = false;
  if constexpr (sizeof(T) == 2) {
    if (latent_mma_shape(dtype, sh)) {
      const int stages = latent_mma_layout(sh.row, 2).total <= kLatentSmemMax ? 2 : 1;
      const size_t smem = latent_mma_layout(sh.row, stages).total;
      const dim3 grid(a.splits, (a.S * sh.H + 15) / 16, a.B);
      static bool done[kMaxDevices] = {};
      if (!done[device]) {
        TSB_CUDA(cudaFuncSetAttribute(latent_attn_mma_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentSmemMax));
        TSB_CUDA(cudaFuncSetAttribute(latent_attn_mma_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentSmemMax));
        TSB_CUDA(cudaFuncSetAttribute(latent_attn_mma_kernel<8>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentSmemMax));
        TSB_CUDA(cudaFuncSetAttribute(latent_attn_mma_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentSmemMax));
        done[device] = true;
      }
      auto k = sh.rank <= 128 ? latent_attn_mma_kernel<2>
                              : (sh.rank <= 256 ? latent_attn_mma_kernel<4> : (sh.rank <= 512 ? latent_attn_mma_kernel<8> : latent_attn_mma_kernel<16>));
      TSB_CUDA(launch_k(k, grid, dim3(kLmThreads), smem, s, sh, a.part, (const bf16*)a.q_lat, (const bf16*)a.cache, a.seq_stride, a.S, a.T0, a.state, a.Tmax,
                        a.splits, stages));
      done_mma = true;
    }
  }
  if (!done_mma) TSB_TRY(latent_simple<T>(device, a, s));
  count_launch(device);
  TSB_CUDA(launch_k(latent_value_kernel<T>, dim3(rows * sh.H, (sh.vdim + kLvCols - 1) / kLvCols), dim3(kLvThreads), (size_t)sh.rank * 4, s, sh, (T*)a.out,
                    (const float*)a.part, (const T*)a.uv, a.splits));
  count_launch(device);
  return check_launch("latent attention");
}

int launch_latent_attention(int device, DeviceState* st, int dtype, const LatentArgs& a, cudaStream_t s) {
  if (a.B == 0 || a.S == 0) return 1;
  const LatentShape& sh = a.shape;
  if (!a.state && latent_expanded(dtype, sh, a.q_stride, a.S)) {
    const int T = a.T0 + a.S, kvw = sh.H * (sh.dim + sh.vdim);
    TSB_CHECK((int64_t)a.B * T * kvw <= a.kv_elems, "latent attention: scratch too small for %d expanded keys", a.B * T);
    for (int b = 0; b < a.B; ++b) {
      Epilogue ep{};
      ep.y = (bf16*)a.kv + (int64_t)b * T * kvw;
      ep.act = TSB200_ACT_NONE;
      TSB_TRY(launch_linear(device, st, dtype, (const bf16*)a.cache + (int64_t)b * a.seq_stride, a.ukv_packed, T, sh.row, kvw, ep, a.lin_ws, a.lin_ws_bytes, s, true));
    }
    const int qk = (sh.dim + sh.rot + 15) / 16 * 16, vn = latent_vn(sh.vdim);
    const size_t smem = latent_prefill_smem(qk, vn);
    const dim3 grid((a.S + kLpRows - 1) / kLpRows, sh.H, a.B);
    static bool done[kMaxDevices] = {};
    if (!done[device]) {
      TSB_CUDA(cudaFuncSetAttribute(latent_prefill_mma_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentSmemMax));
      TSB_CUDA(cudaFuncSetAttribute(latent_prefill_mma_kernel<8>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentSmemMax));
      TSB_CUDA(cudaFuncSetAttribute(latent_prefill_mma_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentSmemMax));
      TSB_CUDA(cudaFuncSetAttribute(latent_prefill_mma_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentSmemMax));
      done[device] = true;
    }
    auto k = vn == 4 ? latent_prefill_mma_kernel<4> : (vn == 8 ? latent_prefill_mma_kernel<8> : (vn == 16 ? latent_prefill_mma_kernel<16> : latent_prefill_mma_kernel<32>));
    k<<<grid, kLpThreads, smem, s>>>(sh, (bf16*)a.out, (const bf16*)a.q, a.q_stride, (const bf16*)a.kv, (const bf16*)a.cache, a.seq_stride, a.S, a.T0, qk);
    count_launch(device);
    return check_launch("latent_prefill_mma");
  }
  if (dtype == TSB200_F32) return latent_absorbed<float>(device, dtype, a, s);
  return latent_absorbed<bf16>(device, dtype, a, s);
}

}  // namespace tsb
