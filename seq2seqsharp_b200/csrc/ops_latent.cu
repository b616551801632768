// Latent attention: the cache keeps one vector per position, [latent c (rank) | rotated key part shared by all heads (rot)], and every
// head's keys and values are linear images of c.  score = (q_n . (Uk_h c) + q_r . k_r) * scale, value = Uv_h c.
//
// Two forms of the same product:
//   absorbed   q_lat = [Uk_h^T q_n | q_r] once per query, then all heads attend to the cache rows themselves (one key of
//              rank + rot elements whose first rank elements are also the value), and Uv_h is applied to the result.  Reads the cache
//              once for all heads: decoding and short portions.
//                latent_query_*          q_lat, and the cache rows of the new positions in CTAs of their own
//                latent_attn_*           the attention, split over the key range
//                latent_value_*          merges the splits and applies Uv_h
//              each as an mma.sync kernel (bf16; in the attention 16 (query, head) rows per CTA, cache rows staged once by cp.async as
//              keys AND values, scores meeting in shared memory so that each warp can own a slice of the latent in the second
//              product) and on CUDA cores (any type and size up to a latent of 1024)
//   expanded   keys and values of all heads are materialised from the cache rows by one tensor-core linear, then causal flash
//              attention per head (latent_prefill_mma_kernel: 128 queries per CTA, mma.sync).  Fewer operations per (query, key)
//              pair, paid for by the expansion: long portions.
// Scores, softmax and sums are fp32 in every kernel; positions and angles come from a table computed in double precision.
#include "kernels.cuh"
#include "warp_tiles.cuh"

namespace tsb {

TSB_CHECKED_WORD(latent)
#ifndef TSB200_CHECKED
int chk_take_latent() { return 0; }
#endif

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
// one cache row from a dkv row, by a whole block: latent norm, rotation of the shared key part
template <typename T>
__device__ __forceinline__ void append_row(const LatentShape& a, const T* x, T* out, const T* norm_w, float eps, const float2* cs, float* red) {
  const int tid = threadIdx.x, nt = blockDim.x, half = a.rot_dims / 2;
  float s = 0.0f;
  for (int i = tid; i < a.rank; i += nt) {
    const float v = to_f<T>(x[i]);
    s += v * v;
  }
  for (int i = tid; i < half; i += nt) turn_pair<T>(x + a.rank, out + a.rank, i, a.rot_dims, cs[i]);
  for (int i = a.rot_dims + tid; i < a.rot; i += nt) out[a.rank + i] = x[a.rank + i];
  s = block_sum(s, red);
  const float inv = 1.0f / sqrtf(s / (float)a.rank + eps);
  for (int i = tid; i < a.rank; i += nt) out[i] = from_f<T>(to_f<T>(x[i]) * inv * to_f<T>(norm_w[i]));
}

struct LatentAppend {   // what the append needs beside the rows
  int dkv_col;          // column of dkv in a q | dkv row; < 0: the layer reads another layer's cache
  const void* norm_w;
  float eps;
  void* cache;
  int64_t seq_stride;
  int S, T0;
  const int* state;
  int Tmax;
  const float2* tab;
};

// rows r0 .. r0 + n - 1 of the batch, one per CTA of the columns blockIdx.x >= H
template <typename T>
__device__ __forceinline__ void append_rows(const LatentShape& a, const T* q, int q_stride, int r0, int n, const LatentAppend& ap, float* red) {
  for (int r = (blockIdx.x - a.H) * gridDim.y + blockIdx.y; r < n; r += (gridDim.x - a.H) * gridDim.y) {
    const int row = r0 + r, b = row / ap.S, pos = state_len(ap.state, b, ap.T0) + row % ap.S;
    TSB_DEV_CHECK(latent, pos >= 0 && pos < ap.Tmax, 0x602, continue)   // append position outside the cache
    if (pos >= ap.Tmax) continue;
    append_row<T>(a, q + (int64_t)row * q_stride + ap.dkv_col, reinterpret_cast<T*>(ap.cache) + (int64_t)b * ap.seq_stride + (int64_t)pos * a.row,
                  (const T*)ap.norm_w, ap.eps, ap.tab + (int64_t)pos * (a.rot_dims / 2), red);
    __syncthreads();
  }
}
// q_lat[row, h, rank ..] = [rotated part | zeros] for n rows, shared out over blockIdx.y
template <typename T>
__device__ __forceinline__ void turn_queries(const LatentShape& a, T* q_lat, const T* q, int q_stride, int h, int r0, int n, const LatentAppend& ap) {
  const int tail = a.row - a.rank, half = a.rot_dims / 2;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < n * tail; i += gridDim.y * blockDim.x) {
    const int r = i / tail, e = i % tail, row = r0 + r;
    const T* x = q + (int64_t)row * q_stride + (int64_t)h * (a.dim + a.rot) + a.dim;
    float v = 0.0f;
    if (e < a.rot_dims) {
      const int pos = min(state_len(ap.state, row / ap.S, ap.T0) + row % ap.S, ap.Tmax - 1);
      const float2 cs = ap.tab[(int64_t)pos * half + (e < half ? e : e - half)];
      v = e < half ? to_f<T>(x[e]) * cs.x - to_f<T>(x[e + half]) * cs.y : to_f<T>(x[e]) * cs.x + to_f<T>(x[e - half]) * cs.y;
    } else if (e < a.rot) {
      v = to_f<T>(x[e]);
    }
    q_lat[((int64_t)row * a.H + h) * a.row + a.rank + e] = from_f<T>(v);
  }
}

// expanded form: queries turned in place, cache rows appended.  grid (rows, 2): y = 0 the query, y = 1 the cache row
constexpr int kLatentAppendThreads = 128;
template <typename T>
__global__ void __launch_bounds__(kLatentAppendThreads) latent_append_kernel(LatentShape a, T* qkv, int row_stride, LatentAppend ap) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x, b = row / ap.S, tid = threadIdx.x;
  const int pos = state_len(ap.state, b, ap.T0) + row % ap.S;
  TSB_DEV_CHECK(latent, pos >= 0 && pos < ap.Tmax, 0x601, return)   // append position outside the cache
  if (pos >= ap.Tmax) return;   // capacity is checked on the host; never write past the cache
  const int half = a.rot_dims / 2;
  const float2* cs = ap.tab + (int64_t)pos * half;
  T* q = qkv + (int64_t)row * row_stride;
  if (blockIdx.y == 0) {
    for (int p = tid; p < a.H * half; p += kLatentAppendThreads) {
      T* r = q + (int64_t)(p / half) * (a.dim + a.rot) + a.dim;
      turn_pair<T>(r, r, p % half, a.rot_dims, cs[p % half]);
    }
  } else {
    append_row<T>(a, q + ap.dkv_col, reinterpret_cast<T*>(ap.cache) + (int64_t)b * ap.seq_stride + (int64_t)pos * a.row, (const T*)ap.norm_w, ap.eps, cs, red);
  }
}

// absorbed form: q_lat[row, h, :] = [sum_d q[row, h, d] Uk[h * dim + d, :] | rotated part | zeros] for eight rows per CTA; the CTAs with
// blockIdx.x >= H append the rows' cache rows
constexpr int kLqThreads = 256, kLqCols = 64, kLqRows = 8;
template <typename T>
__global__ void __launch_bounds__(kLqThreads) latent_query_kernel(LatentShape a, T* q_lat, const T* q, int q_stride, const T* uk, int rows, LatentAppend ap) {
  extern __shared__ float s_q[];              // [8 rows][dim]
  __shared__ float s_red[8][kLqRows][kLqCols];
  pdl_trigger();
  const int h = blockIdx.x, c0 = blockIdx.y * kLqCols, r0 = blockIdx.z * kLqRows;
  const int n = min(kLqRows, rows - r0);
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
  if (h >= a.H) {
    pdl_wait();
    append_rows<T>(a, q, q_stride, r0, n, ap, &s_red[0][0][0]);
    return;
  }
  // this warp's first weights do not depend on the previous kernel
  const int c = c0 + lane * 2;
  const bool in0 = c < a.rank, in1 = c + 1 < a.rank;
  constexpr int PRE = 16;
  float u0[PRE], u1[PRE];
#pragma unroll
  for (int k = 0; k < PRE; ++k) {
    const int dd = w + 8 * k;
    const T* u = uk + ((int64_t)h * a.dim + dd) * a.rank + c;
    u0[k] = u1[k] = 0.0f;
    if (dd < a.dim && in0) {
      if (sizeof(T) == 2 && a.rank % 2 == 0) {
        const float2 t = Pair16<bf16>::get(*reinterpret_cast<const uint32_t*>(u));
        u0[k] = t.x;
        u1[k] = t.y;
      } else {
        u0[k] = to_f<T>(u[0]);
        if (in1) u1[k] = to_f<T>(u[1]);
      }
    }
  }
  pdl_wait();
  const T* qh = q + (int64_t)h * (a.dim + a.rot);
  for (int i = tid; i < kLqRows * a.dim; i += kLqThreads) {
    const int r = i / a.dim;
    s_q[i] = r < n ? to_f<T>(qh[(int64_t)(r0 + r) * q_stride + i % a.dim]) : 0.0f;
  }
  turn_queries<T>(a, q_lat, q, q_stride, h, r0, n, ap);
  __syncthreads();
  float acc[kLqRows][2];
#pragma unroll
  for (int r = 0; r < kLqRows; ++r) acc[r][0] = acc[r][1] = 0.0f;
#pragma unroll
  for (int k = 0; k < PRE; ++k) {
    const int dd = w + 8 * k;
    if (dd < a.dim)
#pragma unroll
      for (int r = 0; r < kLqRows; ++r) {
        acc[r][0] = fmaf(s_q[r * a.dim + dd], u0[k], acc[r][0]);
        acc[r][1] = fmaf(s_q[r * a.dim + dd], u1[k], acc[r][1]);
      }
  }
#pragma unroll 4
  for (int dd = w + 8 * PRE; dd < a.dim; dd += 8) {
    const T* u = uk + ((int64_t)h * a.dim + dd) * a.rank + c;
    const float t0 = in0 ? to_f<T>(u[0]) : 0.0f, t1 = in1 ? to_f<T>(u[1]) : 0.0f;
#pragma unroll
    for (int r = 0; r < kLqRows; ++r) {
      acc[r][0] = fmaf(s_q[r * a.dim + dd], t0, acc[r][0]);
      acc[r][1] = fmaf(s_q[r * a.dim + dd], t1, acc[r][1]);
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

// The same on the warp-level tensor cores: 16 * MT rows and 64 latent columns per CTA, each warp 16 columns.  Uk's tile is requested
// before the wait on the previous kernel.
constexpr int kLqmThreads = 128;
__host__ __device__ inline int latent_q_pitch(int dim) { return (dim + 15) / 16 * 32 + 16; }
template <int MT>
__global__ void __launch_bounds__(kLqmThreads) latent_query_mma_kernel(LatentShape a, bf16* q_lat, const bf16* q, int q_stride, const bf16* uk, int rows,
                                                                       LatentAppend ap) {
  extern __shared__ __align__(128) unsigned char smem[];   // Uk tile [dim to 16][64], query rows [16 MT][dim to 16]
  constexpr int WP = 64 * 2 + 16;
  __shared__ float red[32];
  pdl_trigger();
  const int h = blockIdx.x, c0 = blockIdx.y * 64, r0 = blockIdx.z * 16 * MT, n = min(16 * MT, rows - r0);
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
  if (h >= a.H) {
    pdl_wait();
    append_rows<bf16>(a, q, q_stride, r0, n, ap, red);
    return;
  }
  const int kd = (a.dim + 15) / 16 * 16, qp = latent_q_pitch(a.dim);
  const uint32_t sw = la_smem(smem), sq = sw + kd * WP;
  for (int i = tid; i < kd * 8; i += kLqmThreads) {
    const int k = i >> 3, c = c0 + (i & 7) * 8;
    const bool live = k < a.dim && c < a.rank;
    la_cp16(sw + k * WP + (i & 7) * 16, uk + ((int64_t)h * a.dim + (live ? k : 0)) * a.rank + (live ? c : 0), live);
  }
  pdl_wait();
  const int qc = kd / 8, dc = a.dim / 8;
  for (int r = w; r < 16 * MT; r += kLqmThreads / 32)
    for (int c = lane; c < qc; c += 32) {
      const bool live = r < n && c < dc;
      la_cp16(sq + r * qp + c * 16, q + (int64_t)(r0 + (live ? r : 0)) * q_stride + (int64_t)h * (a.dim + a.rot) + (live ? c : 0) * 8, live);
    }
  la_commit();
  turn_queries<bf16>(a, q_lat, q, q_stride, h, r0, n, ap);
  la_wait<0>();
  __syncthreads();
  float d[MT][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) d[m][i][e] = 0.0f;
  const uint32_t wa = sw + ((lane & 7) + ((lane >> 3) & 1) * 8) * WP + w * 32 + (lane >> 4) * 16;
  const uint32_t aa = sq + (lane & 15) * qp + (lane >> 4) * 16;
#pragma unroll 4
  for (int ks = 0; ks < kd / 16; ++ks) {
    uint32_t b0, b1, b2, b3;
    la_ldsm_x4_trans(wa + ks * 16 * WP, b0, b1, b2, b3);
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      uint32_t a0, a1, a2, a3;
      la_ldsm_x4(aa + m * 16 * qp + ks * 32, a0, a1, a2, a3);
      la_mma(d[m][0], a0, a1, a2, a3, b0, b1);
      la_mma(d[m][1], a0, a1, a2, a3, b2, b3);
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int c = c0 + w * 16 + i * 8 + 2 * t4;
      if (c >= a.rank) continue;   // the latent is a multiple of eight
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = m * 16 + g8 + e * 8;
        if (r < n) *reinterpret_cast<uint32_t*>(q_lat + ((int64_t)(r0 + r) * a.H + h) * a.row + c) = Pair16<bf16>::put(d[m][i][2 * e], d[m][i][2 * e + 1]);
      }
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
  float* out = part + (rr * splits + split) * latent_rec(a.rank);
  for (int e = tid; e < a.rank + 1; e += 256) {   // e = 0: the sum of the weights
    float v = 0.0f;
    for (int q = 0; q < 8; ++q) v += (st[q * rec] == -INFINITY) ? 0.0f : st[q * rec + 1 + e] * expf(st[q * rec] - mx);
    out[e == 0 ? 1 : kRecHead + e - 1] = v;
  }
  if (tid == 0) out[0] = mx;
}

// ---- absorbed form on the warp-level tensor cores -------------------------------------------------------------------------------
constexpr int kLmThreads = 512, kLmKeys = 32, kLmMaxStages = 5;
struct LatentMmaLayout {   // shared memory of latent_attn_mma_kernel
  int pitch;               // bytes of a staged row: an odd number of 16-byte units, so that ldmatrix rows fall into different banks
  uint32_t stage_bytes, s_off, p_off, c_off, total;
};
__host__ __device__ inline LatentMmaLayout latent_mma_layout(int row, int stages) {
  LatentMmaLayout L;
  L.pitch = row * 2 + 16;
  L.stage_bytes = (uint32_t)kLmKeys * L.pitch;
  L.s_off = L.stage_bytes * stages;
  L.p_off = L.s_off + 4 * 16 * (kLmKeys + 4) * 4;
  L.c_off = L.p_off + 16 * (kLmKeys + 8) * 2;
  L.total = L.c_off + 16 * 4;
  return L;
}

// 16 (query, head) rows, sixteen warps, tiles of 32 keys in a ring of 3..5 stages.  Scores: warp w takes keys (w % 4) * 8 .. + 7 and a
// quarter of the inner dimension, its query fragments in registers (KQ steps at most).  Softmax: warp w takes row w, one key per lane.
// Second product: warp w owns NBW * 8 latent columns.  The scores of tile t and the second product of tile t - 1 share an interval between
// two barriers, so a tile costs two of them.
template <int NBW, int KQ>   // NBW even
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
  float* sS = reinterpret_cast<float*>(smem + L.s_off);   // [4 quarters][16][SP]
  bf16* sP = reinterpret_cast<bf16*>(smem + L.p_off);
  float* s_c = reinterpret_cast<float*>(smem + L.c_off);
  constexpr int SP = kLmKeys + 4, PP = kLmKeys + 8, NW = kLmThreads / 32;

  // this thread's share of a tile: chunks lane, lane + 32, ... of the rows w and w + 16
  constexpr int NCH = (KQ * 8 + 31) / 32;
  const bf16* src = base + (int64_t)(t_beg + w) * a.row + lane * 8;
  const uint32_t dst0 = sbase + w * L.pitch + lane * 16;
  uint32_t dst_off = 0;
  const int row16 = NW * a.row;
  int to_issue = 0;                            // tile the next call requests
  auto issue = [&]() {
    if (to_issue < n_tiles) {
      const int t = t_beg + to_issue * kLmKeys + w;
      const bool whole = t - w + kLmKeys <= t_end;
#pragma unroll
      for (int q = 0; q < kLmKeys / NW; ++q) {
        // keys beyond the range re-read its last one; their scores are masked
        const bf16* sr = whole || t + q * NW < t_end ? src + q * row16 : base + (int64_t)(t_end - 1) * a.row + lane * 8;
#pragma unroll
        for (int c = 0; c < NCH; ++c)
          if (lane + c * 32 < cpr) la_cp16(dst0 + dst_off + q * NW * L.pitch + c * 512, sr + c * 256);
      }
      src += kLmKeys * a.row;
      ++to_issue;
      dst_off = dst_off + L.stage_bytes == L.s_off ? 0 : dst_off + L.stage_bytes;
    }
    la_commit();
  };
  const int ahead = stages - 2;                // tiles in flight beside the one being scored and the one before it
  for (int i = 0; i < ahead; ++i) issue();
  const int ksteps = a.row / 16, kq4 = (ksteps + 3) / 4;
  const int kblk = w & 3, ks_beg = (w >> 2) * kq4, ks_n = max(0, min(ksteps - ks_beg, kq4));
  uint32_t qf[KQ][4];
  {
    const bool la = r0 + g8 < R, lb = r0 + g8 + 8 < R;
    const bf16* qa = q_lat + ((int64_t)b * R + r0 + (la ? g8 : 0)) * a.row + ks_beg * 16 + 2 * t4;
    const bf16* qb = q_lat + ((int64_t)b * R + r0 + (lb ? g8 + 8 : 0)) * a.row + ks_beg * 16 + 2 * t4;
#pragma unroll
    for (int k = 0; k < KQ; ++k) {
      qf[k][0] = k < ks_n && la ? *reinterpret_cast<const uint32_t*>(qa + k * 16) : 0u;
      qf[k][1] = k < ks_n && lb ? *reinterpret_cast<const uint32_t*>(qb + k * 16) : 0u;
      qf[k][2] = k < ks_n && la ? *reinterpret_cast<const uint32_t*>(qa + k * 16 + 8) : 0u;
      qf[k][3] = k < ks_n && lb ? *reinterpret_cast<const uint32_t*>(qb + k * 16 + 8) : 0u;
    }
  }
  const uint32_t ka0 = sbase + (kblk * 8 + (lane & 7)) * L.pitch + (lane >> 3) * 16 + ks_beg * 32;
  const uint32_t ka2 = sbase + (kblk * 8 + (lane & 7)) * L.pitch + ((lane >> 3) & 1) * 16 + ks_beg * 32;
  float o[NBW][4];
#pragma unroll
  for (int i = 0; i < NBW; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
  const int col0 = w * NBW * 8;                // first latent column of this warp
  const uint32_t pa = la_smem(sP) + (lane & 15) * (PP * 2) + (lane >> 4) * 16;
  const uint32_t va0 = sbase + ((lane & 7) + ((lane >> 3) & 1) * 8) * L.pitch + (lane >> 4) * 16 + col0 * 2;
  const int row_lim = min(t_end, r0 + w < R ? T0 + (r0 + w) / a.H + 1 : 0);   // softmax row w: keys below are visible to it
  float m_run = -INFINITY, l_run = 0.0f;       // state of row w, the same in every lane

  const bool whole_q = ks_n == KQ, whole_o = col0 + NBW * 8 <= a.rank;
  uint32_t k_off = 0, v_off = 0;               // stages of this tile's keys and of the previous tile's values
  for (int tile = 0; tile <= n_tiles; ++tile) {
    issue();                                   // over the stage of tile - 2, which the previous interval was the last to read
    if (ahead == 3) la_wait<3>();
    else if (ahead == 2) la_wait<2>();
    else la_wait<1>();
    __syncthreads();
    if (tile < n_tiles) {
      const uint32_t ka = ka0 + k_off;
      float c0[4] = {0.0f, 0.0f, 0.0f, 0.0f}, c1[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      if (whole_q) {
        uint32_t kf[KQ + 1][2];
#pragma unroll
        for (int k = 0; k < KQ; k += 2) {
          if (k + 1 < KQ) la_ldsm_x4(ka + k * 32, kf[k][0], kf[k][1], kf[k + 1][0], kf[k + 1][1]);
          else la_ldsm_x2(ka2 + k_off + k * 32, kf[k][0], kf[k][1]);
        }
#pragma unroll
        for (int k = 0; k < KQ; ++k) la_mma(k & 1 ? c1 : c0, qf[k][0], qf[k][1], qf[k][2], qf[k][3], kf[k][0], kf[k][1]);
      } else {
#pragma unroll
        for (int k = 0; k < KQ; k += 2)
          if (k < ks_n) {                      // an odd end also reads the next 32 bytes of shared memory and does not use them
            uint32_t b0, b1, b2, b3;
            la_ldsm_x4(ka + k * 32, b0, b1, b2, b3);
            la_mma(c0, qf[k][0], qf[k][1], qf[k][2], qf[k][3], b0, b1);
            if (k + 1 < KQ && k + 1 < ks_n) la_mma(c1, qf[k + 1 < KQ ? k + 1 : k][0], qf[k + 1 < KQ ? k + 1 : k][1], qf[k + 1 < KQ ? k + 1 : k][2], qf[k + 1 < KQ ? k + 1 : k][3], b2, b3);
          }
      }
      float* d = sS + (w >> 2) * 16 * SP + kblk * 8 + 2 * t4;
      *reinterpret_cast<float2*>(d + g8 * SP) = make_float2(c0[0] + c1[0], c0[1] + c1[1]);
      *reinterpret_cast<float2*>(d + (g8 + 8) * SP) = make_float2(c0[2] + c1[2], c0[3] + c1[3]);
    }
    if (tile > 0 && col0 < a.rank) {
      const float cA = s_c[g8], cB = s_c[g8 + 8];
#pragma unroll
      for (int i = 0; i < NBW; ++i) {
        o[i][0] *= cA; o[i][1] *= cA; o[i][2] *= cB; o[i][3] *= cB;
      }
      const uint32_t va = va0 + v_off;
#pragma unroll
      for (int ks = 0; ks < kLmKeys / 16; ++ks) {
        uint32_t a0, a1, a2, a3;
        la_ldsm_x4(pa + ks * 32, a0, a1, a2, a3);
#pragma unroll
        for (int i = 0; i < NBW; i += 2) {
          if (whole_o || col0 + i * 8 < a.rank) {   // the row is a multiple of 16 elements: both blocks of the pair are inside it
            uint32_t b0, b1, b2, b3;
            la_ldsm_x4_trans(va + ks * 16 * L.pitch + i * 16, b0, b1, b2, b3);
            la_mma(o[i], a0, a1, a2, a3, b0, b1);
            la_mma(o[i + 1], a0, a1, a2, a3, b2, b3);
          }
        }
      }
    }
    __syncthreads();
    if (tile < n_tiles) {
      const int t = t_beg + tile * kLmKeys + lane;
      const float* z4 = sS + w * SP + lane;
      const float z = t < row_lim ? ((z4[0] + z4[16 * SP]) + (z4[32 * SP] + z4[48 * SP])) * a.scale : -INFINITY;
      const float m_new = fmaxf(m_run, warp_max(z));
      const bool none = m_new == -INFINITY;      // the row has seen no key yet
      const float p = none ? 0.0f : __expf(z - m_new), corr = none ? 1.0f : __expf(m_run - m_new);
      sP[w * PP + lane] = from_f<bf16>(p);
      l_run = l_run * corr + warp_sum(p);
      m_run = m_new;
      if (lane == 0) s_c[w] = corr;
    }
    v_off = k_off;
    k_off = k_off + L.stage_bytes == L.s_off ? 0 : k_off + L.stage_bytes;
  }
  la_wait<0>();
  const int rec = latent_rec(a.rank);
  float* pb = part + (((int64_t)b * R + r0) * splits + split) * rec;
#pragma unroll
  for (int i = 0; i < NBW; ++i) {
    const int c = col0 + i * 8 + 2 * t4;
    if (c >= a.rank) continue;   // the latent is a multiple of eight
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int rr = g8 + e * 8;
      if (r0 + rr < R) *reinterpret_cast<float2*>(pb + (int64_t)rr * splits * rec + kRecHead + c) = make_float2(o[i][2 * e], o[i][2 * e + 1]);
    }
  }
  if (lane == 0 && r0 + w < R) {
    pb[(int64_t)w * splits * rec] = m_run;
    pb[(int64_t)w * splits * rec + 1] = l_run;
  }
}

// merges the splits of up to eight rows of one head and applies Uv_h: 32 value elements per CTA, four per warp
constexpr int kLvThreads = 256, kLvCols = 32, kMaxSplits = 64;
template <typename T, int kLvRows>
__global__ void __launch_bounds__(kLvThreads) latent_value_kernel(LatentShape a, T* out, const float* part, const T* uv, int splits, int rows) {
  extern __shared__ float s_o[];   // [8][rank]
  __shared__ float s_w[kLvRows][kMaxSplits];
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, v0 = blockIdx.y * kLvCols, r0 = blockIdx.z * kLvRows;
  const int n = min(kLvRows, rows - r0);
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, rec = latent_rec(a.rank);
  if (w < n) {   // weight of every split of row w
    const float* p = part + ((int64_t)(r0 + w) * a.H + h) * splits * rec;
    const float m0 = lane < splits ? p[(int64_t)lane * rec] : -INFINITY, m1 = lane + 32 < splits ? p[(int64_t)(lane + 32) * rec] : -INFINITY;
    const float l0 = lane < splits ? p[(int64_t)lane * rec + 1] : 0.0f, l1 = lane + 32 < splits ? p[(int64_t)(lane + 32) * rec + 1] : 0.0f;
    const float mx = warp_max(fmaxf(m0, m1));
    const float e0 = m0 == -INFINITY ? 0.0f : expf(m0 - mx), e1 = m1 == -INFINITY ? 0.0f : expf(m1 - mx);
    const float l = warp_sum(l0 * e0 + l1 * e1), inv = l > 0.0f ? 1.0f / l : 0.0f;
    s_w[w][lane] = e0 * inv;
    s_w[w][lane + 32] = e1 * inv;
  }
  __syncthreads();
  for (int i = tid; i < n * a.rank; i += kLvThreads) {
    const int r = kLvRows == 1 ? 0 : i / a.rank, e = i - r * a.rank;
    const float* p = part + ((int64_t)(r0 + r) * a.H + h) * splits * rec + kRecHead + e;
    float v = 0.0f;
#pragma unroll 8
    for (int q = 0; q < splits; ++q) {
      v = fmaf(s_w[r][q], p[(int64_t)q * rec], v);   // an empty split left zeros and has weight 0
    }
    s_o[i] = v;
  }
  __syncthreads();
  float acc[4][kLvRows];
#pragma unroll
  for (int q = 0; q < 4; ++q)
#pragma unroll
    for (int r = 0; r < kLvRows; ++r) acc[q][r] = 0.0f;
  const T* u = uv + ((int64_t)h * a.vdim + v0 + w * 4) * a.rank;
  const int nq = min(4, a.vdim - v0 - w * 4);   // <= 0: this warp's columns do not exist
  bool pairs = false;
  if constexpr (sizeof(T) == 2) pairs = a.rank % 2 == 0;
  if (pairs) {
    if constexpr (sizeof(T) == 2) {
#pragma unroll 2
      for (int e = lane * 2; e < a.rank; e += 64) {
        float2 t[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) t[q] = q < nq ? Pair16<bf16>::get(*reinterpret_cast<const uint32_t*>(u + (int64_t)q * a.rank + e)) : make_float2(0.0f, 0.0f);
#pragma unroll
        for (int r = 0; r < kLvRows; ++r)
          if (r < n) {
            const float2 o = *reinterpret_cast<const float2*>(s_o + r * a.rank + e);
#pragma unroll
            for (int q = 0; q < 4; ++q) acc[q][r] = fmaf(t[q].y, o.y, fmaf(t[q].x, o.x, acc[q][r]));
          }
      }
    }
  } else {
    for (int e = lane; e < a.rank; e += 32) {
      float t[4];
#pragma unroll
      for (int q = 0; q < 4; ++q) t[q] = q < nq ? to_f<T>(u[(int64_t)q * a.rank + e]) : 0.0f;
#pragma unroll
      for (int r = 0; r < kLvRows; ++r)
        if (r < n) {
          const float o = s_o[r * a.rank + e];
#pragma unroll
          for (int q = 0; q < 4; ++q) acc[q][r] = fmaf(t[q], o, acc[q][r]);
        }
    }
  }
#pragma unroll
  for (int r = 0; r < kLvRows; ++r)
    if (r < n) {
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float v = warp_sum(acc[q][r]);
        if (lane == 0 && q < nq) out[((int64_t)(r0 + r) * a.H + h) * a.vdim + v0 + w * 4 + q] = from_f<T>(v);
      }
    }
}

// The same on the warp-level tensor cores: up to 16 rows of one head and 32 value elements per CTA.  Uv's tile is requested before the wait on
// the previous kernel; warp w takes value block w % 4 and every second step of the inner dimension.
__host__ __device__ inline int latent_v_pitch(int rank) { return (rank + 15) / 16 * 32 + 16; }
__global__ void __launch_bounds__(kLvThreads) latent_value_mma_kernel(LatentShape a, bf16* out, const float* part, const bf16* uv, int splits, int rows,
                                                                      int rows_per_cta) {
  extern __shared__ __align__(128) unsigned char smem[];   // Uv tile [32][rank to 16], merged rows [16][rank to 16]
  __shared__ float s_w[16][kMaxSplits];
  __shared__ float4 s_half[4][32];
  pdl_trigger();
  const int h = blockIdx.x, v0 = blockIdx.y * kLvCols, r0 = blockIdx.z * rows_per_cta;
  const int n = min(rows_per_cta, rows - r0);
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, g8 = lane >> 2, t4 = lane & 3, rec = latent_rec(a.rank);
  const int pitch = latent_v_pitch(a.rank), kr = (a.rank + 15) / 16 * 16, chunks = kr / 8, live_chunks = a.rank / 8;
  const uint32_t su = la_smem(smem), so = su + 32 * pitch;
  for (int q = w; q < 32; q += 8)
    for (int c = lane; c < chunks; c += 32) {
      const bool live = v0 + q < a.vdim && c < live_chunks;
      la_cp16(su + q * pitch + c * 16, uv + ((int64_t)h * a.vdim + (live ? v0 + q : 0)) * a.rank + (live ? c : 0) * 8, live);
    }
  la_commit();
  pdl_wait();
  for (int r = w; r < n; r += 8) {   // weight of every split of row r
    const float* p = part + ((int64_t)(r0 + r) * a.H + h) * splits * rec;
    const float m0 = lane < splits ? p[(int64_t)lane * rec] : -INFINITY, m1 = lane + 32 < splits ? p[(int64_t)(lane + 32) * rec] : -INFINITY;
    const float l0 = lane < splits ? p[(int64_t)lane * rec + 1] : 0.0f, l1 = lane + 32 < splits ? p[(int64_t)(lane + 32) * rec + 1] : 0.0f;
    const float mx = warp_max(fmaxf(m0, m1));
    const float e0 = m0 == -INFINITY ? 0.0f : expf(m0 - mx), e1 = m1 == -INFINITY ? 0.0f : expf(m1 - mx);
    const float l = warp_sum(l0 * e0 + l1 * e1), inv = l > 0.0f ? 1.0f / l : 0.0f;
    s_w[r][lane] = e0 * inv;
    s_w[r][lane + 32] = e1 * inv;
  }
  __syncthreads();
  const int half = kr / 2;   // pairs per row
  for (int i = tid; i < (16 - n) * half; i += kLvThreads) *reinterpret_cast<uint32_t*>(smem + (32 + n + i / half) * pitch + (i % half) * 4) = 0u;
  const int64_t split_step = rec / 4, row_step = (int64_t)a.H * splits * split_step;
  const int groups = n <= 2 ? n : (n + 3) / 4;   // four columns of one row (few rows) or of four rows at a time
  const int quads = kr / 4;
  for (int idx = tid; idx < groups * quads; idx += kLvThreads) {
    const int g = idx / quads, e = idx - g * quads;
    const bool live = e * 4 < a.rank;
    if (n <= 2) {
      const float4* p = reinterpret_cast<const float4*>(part + ((int64_t)(r0 + g) * a.H + h) * splits * rec + kRecHead) + e;
      float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      if (live) {
#pragma unroll 8
        for (int q = 0; q < splits; ++q, p += split_step) {
          const float4 t = *p;
          const float f = s_w[g][q];
          x.x = fmaf(f, t.x, x.x); x.y = fmaf(f, t.y, x.y); x.z = fmaf(f, t.z, x.z); x.w = fmaf(f, t.w, x.w);
        }
      }
      *reinterpret_cast<uint2*>(smem + (32 + g) * pitch + e * 8) = make_uint2(Pair16<bf16>::put(x.x, x.y), Pair16<bf16>::put(x.z, x.w));
    } else {
      const int rg = g * 4;
      const float4* p = reinterpret_cast<const float4*>(part + ((int64_t)(r0 + rg) * a.H + h) * splits * rec + kRecHead) + e;
      float4 x[4];
#pragma unroll
      for (int r = 0; r < 4; ++r) x[r] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      if (live) {
#pragma unroll 2
        for (int q = 0; q < splits; ++q, p += split_step)
#pragma unroll
          for (int r = 0; r < 4; ++r)
            if (rg + r < n) {
              const float4 t = p[r * row_step];
              const float f = s_w[rg + r][q];
              x[r].x = fmaf(f, t.x, x[r].x); x[r].y = fmaf(f, t.y, x[r].y); x[r].z = fmaf(f, t.z, x[r].z); x[r].w = fmaf(f, t.w, x[r].w);
            }
      }
#pragma unroll
      for (int r = 0; r < 4; ++r)
        if (rg + r < n) *reinterpret_cast<uint2*>(smem + (32 + rg + r) * pitch + e * 8) = make_uint2(Pair16<bf16>::put(x[r].x, x[r].y), Pair16<bf16>::put(x[r].z, x[r].w));
    }
  }
  la_wait<0>();
  __syncthreads();
  float d0[4] = {0.0f, 0.0f, 0.0f, 0.0f};
  const int nb = w & 3, kh = w >> 2;
  const uint32_t aa = so + (lane & 15) * pitch + (lane >> 4) * 16, ba = su + (nb * 8 + (lane & 7)) * pitch + ((lane >> 3) & 1) * 16;
#pragma unroll 4
  for (int ks = kh; ks < kr / 16; ks += 2) {
    uint32_t a0, a1, a2, a3, b0, b1;
    la_ldsm_x4(aa + ks * 32, a0, a1, a2, a3);
    la_ldsm_x2(ba + ks * 32, b0, b1);
    la_mma(d0, a0, a1, a2, a3, b0, b1);
  }
  if (kh == 1) s_half[nb][lane] = make_float4(d0[0], d0[1], d0[2], d0[3]);
  __syncthreads();
  if (kh == 0) {
    const float4 t = s_half[nb][lane];
    const int c = v0 + nb * 8 + 2 * t4;
    if (c < a.vdim) {   // the value size is even: the pair is inside
      if (g8 < n) *reinterpret_cast<uint32_t*>(out + ((int64_t)(r0 + g8) * a.H + h) * a.vdim + c) = Pair16<bf16>::put(d0[0] + t.x, d0[1] + t.y);
      if (g8 + 8 < n) *reinterpret_cast<uint32_t*>(out + ((int64_t)(r0 + g8 + 8) * a.H + h) * a.vdim + c) = Pair16<bf16>::put(d0[2] + t.z, d0[3] + t.w);
    }
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
        la_mma(sc[0], a0, a1, a2, a3, b0, b1);
        la_mma(sc[1], a0, a1, a2, a3, b2, b3);
        la_ldsm_x4(ka + 16 * qpitch + ks * 32, b0, b1, b2, b3);
        la_mma(sc[2], a0, a1, a2, a3, b0, b1);
        la_mma(sc[3], a0, a1, a2, a3, b2, b3);
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
          la_mma(o[i], p0, p1, p2, p3, b0, b1);
          la_mma(o[i + 1], p0, p1, p2, p3, b2, b3);
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

constexpr size_t kLatentSmemMax = 226 * 1024;
static bool latent_mma_shape(int dtype, const LatentShape& a) {
  return dtype == TSB200_BF16 && a.rank % 8 == 0 && a.rank <= 1024 && a.row <= 17 * 64 && latent_mma_layout(a.row, 3).total <= kLatentSmemMax;
}

// splits of the key range: about one CTA per SM (two with short cache rows, which fit twice), at least 128 keys each
int latent_pick_splits(DeviceState* st, const LatentShape& a, int B, int S, int T) {
  const int64_t base = (int64_t)B * (((int64_t)S * a.H + 15) / 16);
  int64_t n = ((a.row <= 320 ? 2 : 1) * (int64_t)st->sm_count + base / 2) / base;
  const int by_len = (T + 127) / 128;
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

static LatentAppend latent_append_args(const LatentArgs& a) {
  return LatentAppend{a.dkv_col, a.norm_w, a.eps, a.cache, a.seq_stride, a.S, a.T0, a.state, a.Tmax, a.tab};
}

// CTA columns for the append beside the heads': one row per CTA
static int latent_append_columns(const LatentArgs& a, int rows_per_z, int grid_y) {
  if (a.dkv_col < 0) return 0;
  const int rows = a.B * a.S < rows_per_z ? a.B * a.S : rows_per_z;
  return (rows + grid_y - 1) / grid_y;
}

// bf16 shapes whose pieces are multiples of 16 bytes: every kernel of the absorbed form on the tensor cores
static bool latent_mma_pieces(const LatentArgs& a) {
  const LatentShape& sh = a.shape;
  return latent_mma_shape(TSB200_BF16, sh) && sh.dim % 8 == 0 && (sh.dim + sh.rot) % 8 == 0 && a.q_stride % 8 == 0 && sh.vdim % 2 == 0;
}
static int latent_absorbed_mma(int device, DeviceState* st, const LatentArgs& a, cudaStream_t s) {
  const LatentShape& sh = a.shape;
  const int rows = a.B * a.S;
  static bool done[kMaxDevices] = {};
  if (!done[device]) {
    const auto dyn = cudaFuncAttributeMaxDynamicSharedMemorySize;
    TSB_CUDA(cudaFuncSetAttribute(latent_attn_mma_kernel<2, 5>, dyn, (int)kLatentSmemMax));
    TSB_CUDA(cudaFuncSetAttribute(latent_attn_mma_kernel<2, 17>, dyn, (int)kLatentSmemMax));
    TSB_CUDA(cudaFuncSetAttribute(latent_attn_mma_kernel<4, 9>, dyn, (int)kLatentSmemMax));
    TSB_CUDA(cudaFuncSetAttribute(latent_attn_mma_kernel<4, 17>, dyn, (int)kLatentSmemMax));
    TSB_CUDA(cudaFuncSetAttribute(latent_attn_mma_kernel<8, 17>, dyn, (int)kLatentSmemMax));
    TSB_CUDA(cudaFuncSetAttribute(latent_query_mma_kernel<1>, dyn, (int)kLatentSmemMax));
    TSB_CUDA(cudaFuncSetAttribute(latent_query_mma_kernel<4>, dyn, (int)kLatentSmemMax));
    TSB_CUDA(cudaFuncSetAttribute(latent_value_mma_kernel, dyn, 48 * latent_v_pitch(1024)));
    done[device] = true;
  }
  const LatentAppend ap = latent_append_args(a);
  const int kd = (sh.dim + 15) / 16 * 16, mt = rows > 16 ? 4 : 1;
  const size_t sq = (size_t)kd * (64 * 2 + 16) + (size_t)16 * mt * latent_q_pitch(sh.dim);
  TSB_CHECK(sq <= kLatentSmemMax, "latent attention: unrotated head size %d is not supported", sh.dim);
  TSB_CUDA(launch_k(mt == 4 ? latent_query_mma_kernel<4> : latent_query_mma_kernel<1>,
                    dim3(sh.H + latent_append_columns(a, 16 * mt, (sh.rank + 63) / 64), (sh.rank + 63) / 64, (rows + 16 * mt - 1) / (16 * mt)), dim3(kLqmThreads), sq, s, sh, (bf16*)a.q_lat,
                    (const bf16*)a.q, a.q_stride, (const bf16*)a.uk, rows, ap));
  int stages = kLmMaxStages;
  while (stages > 3 && latent_mma_layout(sh.row, stages).total > kLatentSmemMax) --stages;
  const int kq = (sh.row / 16 + 3) / 4;
  auto k = sh.rank <= 256 ? (kq <= 5 ? latent_attn_mma_kernel<2, 5> : latent_attn_mma_kernel<2, 17>)
                          : (sh.rank <= 512 ? (kq <= 9 ? latent_attn_mma_kernel<4, 9> : latent_attn_mma_kernel<4, 17>) : latent_attn_mma_kernel<8, 17>);
  TSB_CUDA(launch_k(k, dim3(a.splits, (a.S * sh.H + 15) / 16, a.B), dim3(kLmThreads), (size_t)latent_mma_layout(sh.row, stages).total, s, sh, a.part,
                    (const bf16*)a.q_lat, (const bf16*)a.cache, a.seq_stride, a.S, a.T0, a.state, a.Tmax, a.splits, stages));
  // few rows: one per CTA, so that the merges run side by side
  const int vt = (sh.vdim + kLvCols - 1) / kLvCols;
  int rt = 1;
  while (rt < 16 && (int64_t)sh.H * vt * ((rows + rt - 1) / rt) > 4 * (int64_t)st->sm_count) ++rt;   // four CTAs fit on an SM: one wave
  TSB_CUDA(launch_k(latent_value_mma_kernel, dim3(sh.H, vt, (rows + rt - 1) / rt), dim3(kLvThreads), (size_t)48 * latent_v_pitch(sh.rank), s, sh, (bf16*)a.out,
                    (const float*)a.part, (const bf16*)a.uv, a.splits, rows, rt));
  count_launch(device, 3);
  return check_launch("latent attention (tensor cores)");
}

// any type and size, CUDA cores
template <typename T>
static int latent_absorbed(int device, DeviceState* st, const LatentArgs& a, cudaStream_t s) {
  const LatentShape& sh = a.shape;
  const int rows = a.B * a.S;
  const size_t sq = (size_t)kLqRows * sh.dim * sizeof(float);
  TSB_CHECK(sq <= 24 * 1024, "latent attention: unrotated head size %d is not supported (at most 768)", sh.dim);
  const LatentAppend ap = latent_append_args(a);
  TSB_CUDA(launch_k(latent_query_kernel<T>, dim3(sh.H + latent_append_columns(a, kLqRows, (sh.rank + kLqCols - 1) / kLqCols), (sh.rank + kLqCols - 1) / kLqCols, (rows + kLqRows - 1) / kLqRows),
                    dim3(kLqThreads), sq, s, sh, (T*)a.q_lat, (const T*)a.q, a.q_stride, (const T*)a.uk, rows, ap));
  TSB_TRY(latent_simple<T>(device, a, s));
  const int vt = (sh.vdim + kLvCols - 1) / kLvCols;   // few rows: one per CTA, so that the merges run side by side; many: eight share a read of Uv
  const int rb = (int64_t)sh.H * vt * rows >= 16 * (int64_t)st->sm_count ? 8 : 1;
  auto k = rb == 8 ? latent_value_kernel<T, 8> : latent_value_kernel<T, 1>;
  TSB_CUDA(launch_k(k, dim3(sh.H, vt, (rows + rb - 1) / rb), dim3(kLvThreads), (size_t)rb * sh.rank * 4, s, sh, (T*)a.out, (const float*)a.part, (const T*)a.uv,
                    a.splits, rows));
  count_launch(device, 3);
  return check_launch("latent attention");
}

int launch_latent_attention(int device, DeviceState* st, int dtype, const LatentArgs& a, cudaStream_t s) {
  if (a.B == 0 || a.S == 0) return 1;
  const LatentShape& sh = a.shape;
  TSB_CHECK(a.state || a.T0 + a.S <= a.Tmax, "latent attention: cache capacity exceeded (%d + %d > %d)", a.T0, a.S, a.Tmax);
  if (!a.state && latent_expanded(dtype, sh, a.q_stride, a.S)) {
    const int T = a.T0 + a.S, kvw = sh.H * (sh.dim + sh.vdim);
    latent_append_kernel<bf16><<<dim3(a.B * a.S, a.dkv_col >= 0 ? 2 : 1), kLatentAppendThreads, 0, s>>>(sh, (bf16*)a.q, a.q_stride, latent_append_args(a));
    count_launch(device);
    TSB_TRY(check_launch("latent_append"));
    TSB_CHECK((int64_t)a.B * T * kvw <= a.kv_elems, "latent attention: scratch too small for %d expanded keys", a.B * T);
    const void* rows = a.cache;
    if (a.B > 1) {   // the sequences' cache rows side by side: one product for the whole batch
      TSB_CHECK((int64_t)a.B * T * sh.row <= a.compact_elems, "latent attention: scratch too small for %d cache rows", a.B * T);
      TSB_CUDA(cudaMemcpy2DAsync(a.compact, (size_t)T * sh.row * 2, a.cache, (size_t)a.seq_stride * 2, (size_t)T * sh.row * 2, a.B, cudaMemcpyDeviceToDevice, s));
      rows = a.compact;
    }
    Epilogue ep{};
    ep.y = a.kv;
    ep.act = TSB200_ACT_NONE;
    TSB_TRY(launch_linear(device, st, dtype, rows, a.ukv_packed, a.B * T, sh.row, kvw, ep, a.lin_ws, a.lin_ws_bytes, s, true));
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
  TSB_CHECK(a.splits >= 1 && a.splits <= kMaxSplits, "latent attention: %d splits", a.splits);
  TSB_CHECK((int64_t)a.B * a.S * sh.H * a.splits * latent_rec(sh.rank) <= a.part_elems, "latent attention: scratch too small for %d rows in %d splits", a.B * a.S, a.splits);
  if (dtype == TSB200_F32) return latent_absorbed<float>(device, st, a, s);
  return latent_mma_pieces(a) ? latent_absorbed_mma(device, st, a, s) : latent_absorbed<bf16>(device, st, a, s);
}

}  // namespace tsb
