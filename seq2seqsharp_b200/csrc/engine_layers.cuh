// Layered engines: models whose layers are described one by one (TSB200LayerDesc) instead of by one shape for all.  Part of
// engine.cu: the same Gpt object, cache manager, slots, snapshots, captured decode step and sampling serve both kinds; this
// file holds what differs - weights, cache rows, scratch and the forward pass.
//
// A layer of gated blocks (residual stream x in fp32):
//   block norm   h1, h2 = two weights on one group-wise RMS norm of x (the previous layer's expert outputs join x here);
//                hc = h1 + short convolution of h1
//   one linear   gate1 = sigmoid(h1 G1 + b1), gate2 = sigmoid(h2 G2 + b2), q | dkv = hc W: three sections of one packed matrix,
//                one launch up to 64 rows
//   attention    latent norm, rotation, cache row (or only the query's rotation when the layer reads another layer's cache), latent
//                attention over the cache rows (ops_latent.cu)
//   out          x += gate1 * (attn W_o)
//   experts      two grouped products over rows sorted by expert; their outputs wait for the next block norm
// A layer of sandwich blocks:
//   sandwich norm  the previous sublayer's output joins x through its own norm and scale; h = norm of the sum
//   one linear     q | k | v | head gates (grouped attention), or q | k | v | output gate and, in fp32, the gates' logits (matrix memory)
//   mixer          grouped attention over the cache (ops_grouped.cu) / matrix memory (ops_memory.cu)
//   out            y = mixed W_o, which waits for the next sandwich norm
//   feed-forward   sandwich norm, gate and up projection with the gated unit in the epilogue, down projection
#pragma once

namespace tsb {

struct LayeredLayer {
  TSB200LayerDesc d;
  LatentShape sh;
  int Nq = 0, Nkv = 0;            // columns of q and dkv (0: the layer reads another layer's cache)
  int ct_gate2 = 0, ct_qkv = 0;   // first column tile of the sections of `fused`
  const float2* tab = nullptr;
  void *norm1 = nullptr, *norm2 = nullptr, *conv_w = nullptr, *g1b = nullptr, *g2b = nullptr;
  void *fused = nullptr, *kv_norm = nullptr, *uk = nullptr, *uv = nullptr, *ukv = nullptr, *wo = nullptr;
  void *up = nullptr, *down = nullptr;   // [experts] packed matrices, columns of `up` are interleaved (gate, up) pairs
  int64_t up_bytes = 0, down_bytes = 0;
  int* table = nullptr;
  void* cache = nullptr;          // [max_batch][max_tokens][row]; null: kv_from's
  void* ring = nullptr;           // [max_batch][taps][d]
  // sandwich blocks
  GroupedShape gs{};
  MemoryShape ms{};
  void *norm1b = nullptr, *scale1 = nullptr, *norm2b = nullptr, *scale2 = nullptr;
  int k_col = -1, v_col = -1, g_col = -1, ct_gates = 0;   // columns of k, v and head gates in a projected row; column tile of the memory's gates
  void *qkv_b = nullptr, *q_norm = nullptr, *k_norm = nullptr, *mem_norm = nullptr, *gates_b = nullptr;
  float *bias = nullptr, *sink = nullptr;   // [H][n_bias] by distance, [H]
  int* bucket = nullptr;          // [n_bias] table row of every distance
  void *cK = nullptr, *cV = nullptr, *mem = nullptr;      // cache rows; memory states [max_batch][memory_state_floats]
  int mixed_cols() const { return d.mixer == TSB200_MIXER_LATENT ? sh.H * sh.vdim : d.heads * d.vdim; }
  RouteLayer routes[2]{};         // host copies of the routing scratch (prompts, captured decode step)
  int route_index = -1;
};

struct Layered {
  TSB200LayeredConfig c;
  std::vector<LayeredLayer> L;
  std::set<std::string> missing;  // weights not given yet
  int n_route = 0, max_experts = 0;
  // scratch, grown on demand (ensure_layered)
  struct Buf { void* p = nullptr; int64_t bytes = 0; };
  Buf hcat, gate1, gate2, qkv, attn, hs, hidden, y, q_lat, part, kv, compact, ws;
  Buf gates, counters, chunks;    // sandwich blocks: gate logits, arrival counters of the decode attention, scratch of the memory's prompt kernels
  // routing scratch, one set for prompts and one for the decode step: a prompt between two steps leaves the captured step valid
  struct Routing { Buf ints, layers; int64_t rows = 0; int block = 0; } routing[2];
};

template <typename TD, typename TS>
__global__ void convert_kernel(TD* dst, const TS* src, int64_t n) {
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) dst[i] = from_f<TD>(to_f<TS>(src[i]));
}
static int convert_into(Gpt* g, void* dst, const void* src, int src_dtype, int64_t n) {
  const int gsz = (int)((n + 255) / 256 < 4096 ? (n + 255) / 256 : 4096);
  if (g->c.dtype == TSB200_BF16 && src_dtype == TSB200_BF16) convert_kernel<<<gsz, 256, 0, g->s>>>((__nv_bfloat16*)dst, (const __nv_bfloat16*)src, n);
  else if (g->c.dtype == TSB200_BF16 && src_dtype == TSB200_F32) convert_kernel<<<gsz, 256, 0, g->s>>>((__nv_bfloat16*)dst, (const float*)src, n);
  else if (g->c.dtype == TSB200_F32 && src_dtype == TSB200_BF16) convert_kernel<<<gsz, 256, 0, g->s>>>((float*)dst, (const __nv_bfloat16*)src, n);
  else if (g->c.dtype == TSB200_F32 && src_dtype == TSB200_F32) convert_kernel<<<gsz, 256, 0, g->s>>>((float*)dst, (const float*)src, n);
  else TSB_FAIL("layered engine: weights are F32 or BF16 tensors");
  count_launch(g->c.device);
  return check_launch("convert");
}

static int to_f32(Gpt* g, float* dst, const void* src, int src_dtype, int64_t n) {
  const int gsz = (int)((n + 255) / 256 < 4096 ? (n + 255) / 256 : 4096);
  if (src_dtype == TSB200_BF16) convert_kernel<<<gsz, 256, 0, g->s>>>(dst, (const __nv_bfloat16*)src, n);
  else convert_kernel<<<gsz, 256, 0, g->s>>>(dst, (const float*)src, n);
  count_launch(g->c.device);
  return check_launch("convert");
}
struct LayerDescView {   // rows of the projections of a sandwich block's mixer
  const TSB200LayerDesc& l;
  int kv_heads() const { return l.mixer == TSB200_MIXER_GROUPED ? l.kv_heads : l.heads; }
  int q() const { return l.heads * l.dim; }
  int k() const { return kv_heads() * l.dim; }
  int v() const { return kv_heads() * l.vdim; }
  int o() const { return l.heads * l.vdim; }
};
// Table row of distance n: single distances below rows / 2, then logarithmic up to `far`.
static int distance_bucket(int n, int rows, int far) {
  const int half = rows / 2;
  if (n < half || half < 1) return std::min(n, rows - 1);
  const double at = std::log((double)n / half) / std::log((double)far / half) * (rows - half);
  return std::min<int64_t>(rows - 1, half + (int64_t)std::floor(at));
}

// Every weight of the model by name with its shape ([out, in] for matrices); "table" tensors are int32.
static std::vector<std::pair<std::string, std::pair<int64_t, int64_t>>> layered_weights(const Layered* ly) {
  std::vector<std::pair<std::string, std::pair<int64_t, int64_t>>> v;
  const int64_t d = ly->c.d, V = ly->c.V;
  auto add = [&](const std::string& n, int64_t r, int64_t c) { v.push_back({n, {r, c}}); };
  add("embed", V, d);
  add("final_norm", 1, d);
  if (!ly->c.tied_head) add("head", V, d);
  for (size_t i = 0; i < ly->L.size(); ++i) {
    const LayeredLayer& L = ly->L[i];
    const std::string p = "layer." + std::to_string(i) + ".";
    if (ly->c.block == TSB200_BLOCK_SANDWICH) {
      for (const char* n : {"norm1", "norm1b", "scale1"}) add(p + n, 1, d);
      const int64_t H = L.d.heads, G = L.d.kv_heads, dim = L.d.dim, vdim = L.d.vdim;
      const std::string m = p + (L.d.mixer == TSB200_MIXER_GROUPED ? "attn." : "mem.");
      add(m + "q", H * dim, d);
      if (L.d.mixer == TSB200_MIXER_GROUPED) {
        const bool own = L.d.kv_from < 0;
        if (own) {
          add(m + "k", G * dim, d);
          add(m + "v", G * vdim, d);
        }
        if (L.d.flags & TSB200_ATTN_QKV_BIAS) {
          add(m + "q.b", 1, H * dim);
          if (own) add(m + "k.b", 1, G * dim);
          if (own) add(m + "v.b", 1, G * vdim);
        }
        if (L.d.flags & TSB200_ATTN_QK_NORM) {
          add(m + "q_norm", 1, dim);
          if (own) add(m + "k_norm", 1, dim);
        }
        if (L.d.bias_rows > 0) add(m + "bias", L.d.bias_rows, H);
        if (L.d.flags & TSB200_ATTN_SINK) add(m + "sink", 1, H);
        if (L.d.flags & TSB200_ATTN_HEAD_GATE) add(m + "gate", H, d);
      } else {
        add(m + "k", H * dim, d);
        add(m + "v", H * vdim, d);
        add(m + "gate", H * vdim, d);
        for (const char* n : {"i", "f"}) {
          add(m + n, H, d);
          add(m + n + ".b", 1, H);
        }
        add(m + "norm", 1, H * vdim);
      }
      add(m + "o", d, H * vdim);
      if (L.d.ff > 0) {
        for (const char* n : {"norm2", "norm2b", "scale2"}) add(p + n, 1, d);
        add(p + "ff.gate", L.d.ff, d);
        add(p + "ff.up", L.d.ff, d);
        add(p + "ff.down", d, L.d.ff);
      }
      continue;
    }
    add(p + "norm1", 1, d);
    add(p + "conv1", d, ly->c.conv_taps);
    add(p + "gate1.w", d, d);
    add(p + "gate1.b", 1, d);
    add(p + "attn.q", L.Nq, d);
    if (L.Nkv) {
      add(p + "attn.dkv", L.Nkv, d);
      add(p + "attn.dkv_norm", 1, L.sh.rank);
    }
    add(p + "attn.uk", (int64_t)L.sh.H * L.sh.dim, L.sh.rank);
    add(p + "attn.uv", (int64_t)L.sh.H * L.sh.vdim, L.sh.rank);
    add(p + "attn.o", d, (int64_t)L.sh.H * L.sh.vdim);
    if (L.d.experts > 0) {
      add(p + "norm2", 1, d);
      add(p + "gate2.w", d, d);
      add(p + "gate2.b", 1, d);
      add(p + "experts.table", V, L.d.top);
      for (int e = 0; e < L.d.experts; ++e) {
        const std::string q = p + "experts." + std::to_string(e) + ".";
        add(q + "gate", L.d.ff, d);
        add(q + "up", L.d.ff, d);
        add(q + "down", d, L.d.ff);
      }
    }
  }
  return v;
}

// One weight from device memory (src) into its place(s).
static int layered_put(Gpt* g, const std::string& name, const void* src, int dt, int64_t rows, int64_t cols) {
  Layered* ly = g->ly;
  const int dev = g->c.device, T = g->c.dtype, d = ly->c.d;
  const int64_t n = rows * cols;
  auto pack = [&](void* dst, int N, int K, int Kp, int c0, int cs) {   // [N, K] (out x in) -> columns c0 + j cs of a packed [Kp, ..] matrix
    return launch_pack(dev, g->st, T, dst, dt, src, K, N, K, Kp, c0, cs, g->s, true);
  };
  if (name == "embed") {
    TSB_TRY(convert_into(g, g->E, src, dt, n));
    return !ly->c.tied_head ? 1 : pack(g->head_w, ly->c.V, d, d, 0, 1);
  }
  if (name == "head") return pack(g->head_w, ly->c.V, d, d, 0, 1);
  if (name == "final_norm") return convert_into(g, g->nf_g, src, dt, n);
  int i = -1, used = 0;
  TSB_CHECK(std::sscanf(name.c_str(), "layer.%d.%n", &i, &used) == 1 && used > 0 && i >= 0 && i < (int)ly->L.size(), "unknown weight name '%s'", name.c_str());
  LayeredLayer& L = ly->L[i];
  const std::string f = name.substr(used);
  const int NT = packed_tile_cols(T);
  if (f == "norm1") return convert_into(g, L.norm1, src, dt, n);
  if (f == "norm2") return convert_into(g, L.norm2, src, dt, n);
  if (ly->c.block == TSB200_BLOCK_SANDWICH) {
    const LayerDescView v{L.d};
    auto at = [&](void* base, int64_t elems) { return (void*)((char*)base + elems * (int64_t)dtype_size(T)); };
    if (f == "norm1b") return convert_into(g, L.norm1b, src, dt, n);
    if (f == "scale1") return convert_into(g, L.scale1, src, dt, n);
    if (f == "norm2b") return convert_into(g, L.norm2b, src, dt, n);
    if (f == "scale2") return convert_into(g, L.scale2, src, dt, n);
    if (f == "ff.gate") return pack(L.up, L.d.ff, d, d, 0, 2);
    if (f == "ff.up") return pack(L.up, L.d.ff, d, d, 1, 2);
    if (f == "ff.down") return pack(L.down, d, L.d.ff, L.d.ff, 0, 1);
    if (f == "attn.q" || f == "mem.q") return pack(L.fused, v.q(), d, d, 0, 1);
    if (f == "attn.k" || f == "mem.k") return pack(L.fused, v.k(), d, d, L.k_col, 1);
    if (f == "attn.v" || f == "mem.v") return pack(L.fused, v.v(), d, d, L.v_col, 1);
    if (f == "attn.gate" || f == "mem.gate") return pack(L.fused, L.d.mixer == TSB200_MIXER_GROUPED ? L.d.heads : v.o(), d, d, L.g_col, 1);
    if (f == "attn.o" || f == "mem.o") return pack(L.wo, d, v.o(), v.o(), 0, 1);
    if (f == "attn.q.b") return convert_into(g, L.qkv_b, src, dt, n);
    if (f == "attn.k.b") return convert_into(g, at(L.qkv_b, L.k_col), src, dt, n);
    if (f == "attn.v.b") return convert_into(g, at(L.qkv_b, L.v_col), src, dt, n);
    if (f == "attn.q_norm") return convert_into(g, L.q_norm, src, dt, n);
    if (f == "attn.k_norm") return convert_into(g, L.k_norm, src, dt, n);
    if (f == "attn.bias") return launch_expand_bias(dev, dt, L.bias, src, L.bucket, L.gs.n_bias, L.d.heads, g->s);
    if (f == "attn.sink") return to_f32(g, L.sink, src, dt, n);
    if (f == "mem.i") return pack(L.fused, L.d.heads, d, d, L.ct_gates * NT, 1);
    if (f == "mem.f") return pack(L.fused, L.d.heads, d, d, L.ct_gates * NT + L.d.heads, 1);
    if (f == "mem.i.b") return convert_into(g, L.gates_b, src, dt, n);
    if (f == "mem.f.b") return convert_into(g, at(L.gates_b, L.d.heads), src, dt, n);
    if (f == "mem.norm") return convert_into(g, L.mem_norm, src, dt, n);
    TSB_FAIL("unknown weight name '%s'", name.c_str());
  }
  if (f == "conv1") return convert_into(g, L.conv_w, src, dt, n);
  if (f == "gate1.w") return pack(L.fused, d, d, d, 0, 1);
  if (f == "gate1.b") return convert_into(g, L.g1b, src, dt, n);
  if (f == "gate2.w") return pack(L.fused, d, d, d, L.ct_gate2 * NT, 1);
  if (f == "gate2.b") return convert_into(g, L.g2b, src, dt, n);
  if (f == "attn.q") return pack(L.fused, L.Nq, d, d, L.ct_qkv * NT, 1);
  if (f == "attn.dkv") return pack(L.fused, L.Nkv, d, d, L.ct_qkv * NT + L.Nq, 1);
  if (f == "attn.dkv_norm") return convert_into(g, L.kv_norm, src, dt, n);
  if (f == "attn.uk") {
    TSB_TRY(convert_into(g, L.uk, src, dt, n));
    return pack(L.ukv, L.sh.H * L.sh.dim, L.sh.rank, L.sh.row, 0, 1);
  }
  if (f == "attn.uv") {
    TSB_TRY(convert_into(g, L.uv, src, dt, n));
    return pack(L.ukv, L.sh.H * L.sh.vdim, L.sh.rank, L.sh.row, L.sh.H * L.sh.dim, 1);
  }
  if (f == "attn.o") return pack(L.wo, d, L.sh.H * L.sh.vdim, L.sh.H * L.sh.vdim, 0, 1);
  if (f == "experts.table") {
    TSB_CUDA(cudaMemcpyAsync(L.table, src, (size_t)n * 4, cudaMemcpyDeviceToDevice, g->s));
    return 1;
  }
  int e = -1, at = 0;
  TSB_CHECK(std::sscanf(f.c_str(), "experts.%d.%n", &e, &at) == 1 && at > 0 && e >= 0 && e < L.d.experts, "unknown weight name '%s'", name.c_str());
  const std::string w = f.substr(at);
  if (w == "gate") return pack((char*)L.up + e * L.up_bytes, L.d.ff, d, d, 0, 2);
  if (w == "up") return pack((char*)L.up + e * L.up_bytes, L.d.ff, d, d, 1, 2);
  if (w == "down") return pack((char*)L.down + e * L.down_bytes, d, L.d.ff, L.d.ff, 0, 1);
  TSB_FAIL("unknown weight name '%s'", name.c_str());
}

static int layered_check_table(const LayeredLayer& L, const int32_t* t, int64_t rows) {
  for (int64_t r = 0; r < rows; ++r)
    for (int j = 0; j < L.d.top; ++j)
      TSB_CHECK(t[r * L.d.top + j] >= 0 && t[r * L.d.top + j] < L.d.experts, "expert table: entry %d of token %lld names expert %d of %d", j, (long long)r,
                t[r * L.d.top + j], L.d.experts);
  return 1;
}

static int layered_set_weight(Gpt* g, const char* name, const void* data, int dtype, int64_t rows, int64_t cols, int on_device) {
  Layered* ly = g->ly;
  int64_t er = 0, ec = 0;
  for (auto& w : layered_weights(ly))
    if (w.first == name) {
      er = w.second.first;
      ec = w.second.second;
      break;
    }
  TSB_CHECK(er > 0, "unknown weight name '%s'", name);
  TSB_CHECK(rows == er && cols == ec, "gpt_set_weight: '%s' expects [%lld, %lld], got [%lld, %lld]", name, (long long)er, (long long)ec, (long long)rows,
            (long long)cols);
  const bool table = ends_with(name, "experts.table");
  TSB_CHECK(table ? dtype == TSB200_I32 : (dtype == TSB200_F32 || dtype == TSB200_BF16), "gpt_set_weight: '%s' has an unsupported element type", name);
  const int64_t bytes = rows * cols * (int64_t)dtype_size(dtype);
  if (table) {
    std::vector<int32_t> host;
    const int32_t* t = (const int32_t*)data;
    if (on_device) {
      host.resize((size_t)(rows * cols));
      TSB_CUDA(cudaMemcpy(host.data(), data, (size_t)bytes, cudaMemcpyDeviceToHost));
      t = host.data();
    }
    int i = -1;
    std::sscanf(name, "layer.%d.", &i);
    TSB_TRY(layered_check_table(ly->L[i], t, rows));
  }
  const void* src = data;
  void* tmp = nullptr;
  if (!on_device) {
    cudaError_t e = cudaMalloc(&tmp, (size_t)bytes);
    if (e != cudaSuccess) {
      cudaGetLastError();
      TSB_FAIL("OOM: staging buffer of %lld bytes: %s", (long long)bytes, cudaGetErrorString(e));
    }
    if (cudaMemcpyAsync(tmp, data, (size_t)bytes, cudaMemcpyHostToDevice, g->s) != cudaSuccess) {
      cudaFree(tmp);
      TSB_FAIL("gpt_set_weight: host to device copy failed: %s", cudaGetErrorString(cudaGetLastError()));
    }
    src = tmp;
  }
  int ok = layered_put(g, name, src, dtype, rows, cols);
  if (cudaStreamSynchronize(g->s) != cudaSuccess && ok) {
    set_last_error("gpt_set_weight: %s", cudaGetErrorString(cudaGetLastError()));
    ok = 0;
  }
  if (tmp) cudaFree(tmp);
  if (ok) ly->missing.erase(name);
  return ok;
}

// matrices N(0, std), biases N(0, bias_std), norm gains and scales 1, tables by a hash of (token, choice)
static int layered_fill_synthetic(Gpt* g, uint64_t seed, float std, float bias_std) {
  Layered* ly = g->ly;
  int64_t most = 1;
  const auto all = layered_weights(ly);
  for (auto& w : all) most = std::max(most, w.second.first * w.second.second);
  void* tmp = nullptr;
  if (cudaMalloc(&tmp, (size_t)most * 4) != cudaSuccess) {
    cudaGetLastError();
    TSB_FAIL("OOM: synthetic staging buffer of %lld bytes", (long long)most * 4);
  }
  int ok = 1;
  std::vector<int32_t> host;
  for (auto& w : all) {
    const std::string& n = w.first;
    const int64_t r = w.second.first, c = w.second.second;
    int dt = TSB200_F32;
    if (ends_with(n, "experts.table")) {
      int i = -1;
      std::sscanf(n.c_str(), "layer.%d.", &i);
      const uint64_t E = (uint64_t)ly->L[i].d.experts;
      host.resize((size_t)(r * c));
      for (int64_t t = 0; t < r; ++t) {
        uint64_t h = (seed + 0x9E3779B97F4A7C15ull * (uint64_t)(t + 1) + (uint64_t)i * 0xBF58476D1CE4E5B9ull);
        h = (h ^ (h >> 30)) * 0xBF58476D1CE4E5B9ull;
        h = (h ^ (h >> 27)) * 0x94D049BB133111EBull;
        for (int64_t j = 0; j < c; ++j) host[(size_t)(t * c + j)] = (int32_t)(((h >> 8) + (uint64_t)j) % E);   // neighbours: the entries of a row differ
      }
      dt = TSB200_I32;
      ok = cudaMemcpyAsync(tmp, host.data(), host.size() * 4, cudaMemcpyHostToDevice, g->s) == cudaSuccess;
      if (!ok) set_last_error("gpt_fill_synthetic: table upload failed");
    } else if (n.find("norm") != std::string::npos || n.find(".scale") != std::string::npos) {
      fill_const_kernel<float><<<(int)((r * c + 255) / 256), 256, 0, g->s>>>((float*)tmp, r * c, 1.0f);
    } else {
      const bool bias = ends_with(n, ".b");
      if (bias && bias_std <= 0.0f) ok = cudaMemsetAsync(tmp, 0, (size_t)(r * c) * 4, g->s) == cudaSuccess;
      else ok = launch_synthetic(g->c.device, g->st, tmp, TSB200_F32, r * c, seed, fnv1a64(n.c_str()), bias ? bias_std : std, g->s);
    }
    ok = ok && layered_put(g, n, tmp, dt, r, c);
    if (!ok) break;
    ly->missing.erase(n);
    if (dt == TSB200_I32) cudaStreamSynchronize(g->s);   // `host` is reused
  }
  if (cudaStreamSynchronize(g->s) != cudaSuccess && ok) {
    set_last_error("gpt_fill_synthetic: %s", cudaGetErrorString(cudaGetLastError()));
    ok = 0;
  }
  cudaFree(tmp);
  if (g->gexec) { cudaGraphExecDestroy(g->gexec); g->gexec = nullptr; }
  return ok;
}

static int layered_block_rows(const Layered* ly, int rows) {
  if (rows > 64) return 128;
  int64_t picks = 0, experts = 1;
  for (auto& L : ly->L)
    if (L.d.experts > 0 && (int64_t)rows * L.d.top * experts > picks * L.d.experts) {
      picks = (int64_t)rows * L.d.top;
      experts = L.d.experts;
    }
  return picks > 4 * experts ? 16 : 8;
}
static int layered_max_blocks(int64_t picks, int experts, int block_rows) { return (int)(std::min<int64_t>(picks, experts) + picks / block_rows); }

static int grow(Gpt* g, Layered::Buf& b, int64_t bytes, bool zero = false) {
  if (bytes <= b.bytes) return 1;
  if (b.p) TSB_TRY(dev_free(g, b.p));
  b.p = nullptr;
  b.bytes = 0;
  TSB_TRY(dev_alloc(g, &b.p, bytes, zero));
  b.bytes = bytes;
  // the captured decode step holds the old buffer as a kernel argument
  if (g->gexec) { cudaGraphExecDestroy(g->gexec); g->gexec = nullptr; }
  return 1;
}

static int grow_residual(Gpt* g, int64_t bytes) {
  if (bytes <= g->x_bytes) return 1;
  TSB_CUDA(cudaStreamSynchronize(g->s));
  if (g->x) TSB_TRY(dev_free(g, g->x));
  g->x = nullptr;
  g->x_bytes = 0;
  TSB_TRY(dev_alloc(g, (void**)&g->x, bytes, false));
  g->x_bytes = bytes;
  if (g->gexec) { cudaGraphExecDestroy(g->gexec); g->gexec = nullptr; }
  return 1;
}

static int ensure_sandwich(Gpt* g, int B, int S, int T) {
  Layered* ly = g->ly;
  const int64_t rows = (int64_t)B * S, d = ly->c.d, es = g->es;
  const int dt = g->c.dtype;
  int64_t nq = 0, na = 0, nhid = 0, nqn = 0, npart = 0, ngates = 0, ncnt = 0, nchunk = 0, ws = kWsCounterBytes + 1024;
  auto lin = [&](int64_t K, int64_t N) {
    for (int64_t m : {(int64_t)1, std::min<int64_t>(rows, 64)}) {
      ws = std::max(ws, linear_workspace_bytes((int)m, (int)K, (int)N));
      if (is_16bit(dt)) ws = std::max(ws, gemm_stream_sections_workspace_bytes((int)m, (int)K, (int)N, g->st->sm_count));
    }
  };
  lin(d, ly->c.V);
  for (auto& L : ly->L) {
    const int64_t out = L.mixed_cols();
    nq = std::max(nq, rows * L.Nq);
    na = std::max(na, rows * out);
    if (L.d.mixer == TSB200_MIXER_GROUPED) {
      nqn = std::max(nqn, rows * L.gs.H * L.gs.dk);
      if (S == 1) npart = std::max(npart, grouped_part_elems(L.gs, B, grouped_pick_splits(g->st, dt, L.gs, B, T)));
      ncnt = std::max(ncnt, (int64_t)B * L.gs.H);
      lin(d, L.Nq);
    } else {
      ngates = std::max(ngates, rows * 2 * L.ms.H);
      nchunk = std::max(nchunk, memory_scratch_bytes(dt, L.ms, B, S));
      lin(d, L.Nq + 512 + 2 * L.ms.H);
    }
    lin(out, d);
    if (L.d.ff > 0) {
      nhid = std::max(nhid, rows * L.d.ff);
      lin(d, 2 * L.d.ff);
      lin(L.d.ff, d);
    }
  }
  if (is_16bit(dt)) ws = std::max<int64_t>(ws, 64LL << 20);   // split-K partials of the tensor-core GEMM
  TSB_TRY(grow_residual(g, rows * d * 4));
  TSB_TRY(grow(g, ly->hcat, rows * d * es));
  TSB_TRY(grow(g, ly->y, rows * d * es));
  TSB_TRY(grow(g, ly->qkv, nq * es));
  TSB_TRY(grow(g, ly->attn, na * es));
  TSB_TRY(grow(g, ly->hidden, nhid * es));
  TSB_TRY(grow(g, ly->q_lat, nqn * es));
  TSB_TRY(grow(g, ly->part, npart * 4));
  TSB_TRY(grow(g, ly->gates, ngates * 4));
  TSB_TRY(grow(g, ly->counters, ncnt * 4, true));
  TSB_TRY(grow(g, ly->chunks, nchunk));
  return grow(g, ly->ws, ws, true);
}

// Scratch of a forward pass over B sequences of S new positions on up to T cached ones (T: after the pass); step: for the decode step.
static int ensure_layered(Gpt* g, int B, int S, int T, bool step) {
  Layered* ly = g->ly;
  if (ly->c.block == TSB200_BLOCK_SANDWICH) return ensure_sandwich(g, B, S, T);
  const int64_t rows = (int64_t)B * S, d = ly->c.d, es = g->es;
  const int dt = g->c.dtype;
  const int br = layered_block_rows(ly, (int)rows);
  int64_t nq = 0, na = 0, npk = 0, nhid = 0, nlat = 0, npart = 0, nkv = 0, ncomp = 0, nints = 0;
  int64_t ws = kWsCounterBytes + 1024;
  auto lin = [&](int64_t K, int64_t N) {
    for (int64_t m : {(int64_t)1, std::min<int64_t>(rows, 64)}) {
      ws = std::max(ws, linear_workspace_bytes((int)m, (int)K, (int)N));
      if (is_16bit(dt)) ws = std::max(ws, gemm_stream_mma_workspace_bytes((int)m, (int)K, (int)N, g->st->sm_count));
    }
  };
  lin(d, ly->c.V);
  for (auto& L : ly->L) {
    nq = std::max(nq, rows * (L.Nq + L.Nkv));
    na = std::max(na, rows * L.sh.H * L.sh.vdim);
    if (!latent_expanded(dt, L.sh, L.Nq + L.Nkv, S)) {
      nlat = std::max(nlat, rows * L.sh.H * L.sh.row);
      npart = std::max(npart, rows * L.sh.H * latent_pick_splits(g->st, L.sh, B, S, T) * latent_rec(L.sh.rank));
    } else {
      nkv = std::max(nkv, (int64_t)B * T * L.sh.H * (L.sh.dim + L.sh.vdim));
      if (B > 1) ncomp = std::max(ncomp, (int64_t)B * T * L.sh.row);
      for (int64_t m : {(int64_t)16, (int64_t)64})
        ws = std::max(ws, gemm_stream_mma_workspace_bytes((int)m, L.sh.row, L.sh.H * (L.sh.dim + L.sh.vdim), g->st->sm_count));
    }
    if (is_16bit(dt)) ws = std::max(ws, gemm_stream_sections_workspace_bytes((int)std::min<int64_t>(rows, 64), (int)d, (int)(2 * d + L.Nq + L.Nkv), g->st->sm_count));
    lin(d, d);
    lin(d, L.Nq + L.Nkv);
    lin(L.sh.H * L.sh.vdim, d);
    if (L.d.experts > 0) {
      const int64_t p = rows * L.d.top;
      npk = std::max(npk, p);
      nhid = std::max(nhid, p * L.d.ff);
      const int mb = layered_max_blocks(p, L.d.experts, br);
      nints += 2 * p + 4 * (int64_t)mb + 16;
      if (is_16bit(dt) && br <= 16) {
        ws = std::max(ws, gemm_stream_grouped_workspace_bytes(br, 2 * L.d.ff, mb, g->st->sm_count));
        ws = std::max(ws, gemm_stream_grouped_workspace_bytes(br, (int)d, mb, g->st->sm_count));
      }
    }
  }
  if (is_16bit(dt)) ws = std::max<int64_t>(ws, 64LL << 20);   // split-K partials of the tensor-core GEMM
  TSB_TRY(grow_residual(g, rows * d * 4));
  TSB_TRY(grow(g, ly->hcat, 3 * rows * d * es));
  TSB_TRY(grow(g, ly->gate1, rows * d * es));
  TSB_TRY(grow(g, ly->gate2, rows * d * es));
  TSB_TRY(grow(g, ly->qkv, nq * es));
  TSB_TRY(grow(g, ly->attn, na * es));
  TSB_TRY(grow(g, ly->hs, npk * d * es));
  TSB_TRY(grow(g, ly->hidden, nhid * es));
  TSB_TRY(grow(g, ly->y, npk * d * es));
  TSB_TRY(grow(g, ly->q_lat, nlat * es));
  TSB_TRY(grow(g, ly->part, npart * 4));
  TSB_TRY(grow(g, ly->kv, nkv * es));
  TSB_TRY(grow(g, ly->compact, ncomp * es));
  TSB_TRY(grow(g, ly->ws, ws, true));
  Layered::Routing& rt = ly->routing[step ? 1 : 0];
  if (ly->n_route > 0 && (rt.rows != rows || rt.block != br)) {
    // routing scratch of every expert layer, laid out for this many rows; the captured step holds pointers into its set
    TSB_TRY(grow(g, rt.ints, nints * 4 + 64));
    TSB_TRY(grow(g, rt.layers, (int64_t)ly->n_route * sizeof(RouteLayer)));
    if (step && g->gexec) { cudaGraphExecDestroy(g->gexec); g->gexec = nullptr; }
    std::vector<RouteLayer> host((size_t)ly->n_route);
    int* at = (int*)rt.ints.p;
    for (auto& L : ly->L) {
      if (L.d.experts <= 0) continue;
      const int64_t p = rows * L.d.top;
      RouteLayer& r = L.routes[step ? 1 : 0];
      r.table = L.table;
      r.top = L.d.top;
      r.experts = L.d.experts;
      r.blocks = (RowBlock*)at;   // 16-byte aligned: every piece is a multiple of four ints
      at += 4 * (int64_t)layered_max_blocks(p, L.d.experts, br);
      r.n_blocks = at;
      at += 4;
      r.pos = at;
      at += (p + 3) / 4 * 4;
      r.matrix_of = at;
      at += (p + 3) / 4 * 4;
      host[(size_t)L.route_index] = r;
    }
    TSB_CUDA(cudaMemcpyAsync(rt.layers.p, host.data(), host.size() * sizeof(RouteLayer), cudaMemcpyHostToDevice, g->s));
    TSB_CUDA(cudaStreamSynchronize(g->s));   // `host` is pageable
    rt.rows = rows;
    rt.block = br;
  }
  return 1;
}

// What the layers leave for the final norm: a sublayer output that has not joined the residual yet.
struct LayerPass {
  int B, S, T0, T_plan;
  bool use_state;
  const LayeredLayer* last;
};

static void gated_pending(const Layered* ly, const LayeredLayer* prev, bool use_state, BlockNormArgs& a) {
  if (!prev) return;
  const RouteLayer& r = prev->routes[use_state ? 1 : 0];
  a.y = ly->y.p;
  a.y_pos = r.pos;
  a.top = prev->d.top;
  a.y_gate = ly->gate2.p;
}

// Layers of gated blocks; the last layer's expert outputs stay pending.
static int gated_layers(Gpt* g, LayerPass& ps) {
  Layered* ly = g->ly;
  const int B = ps.B, S = ps.S, T0 = ps.T0, T_plan = ps.T_plan;
  const bool use_state = ps.use_state;
  const int dev = g->c.device, dt = g->c.dtype, d = ly->c.d, rows = B * S;
  const int64_t es = g->es;
  const int* dT = use_state ? g->state : nullptr;
  const bool pdl = g->pdl;
  const Layered::Routing& rt = ly->routing[use_state ? 1 : 0];
  auto route_of = [&](const LayeredLayer& L) -> const RouteLayer& { return L.routes[use_state ? 1 : 0]; };
  void *ws = ly->ws.p;
  const int64_t wsb = ly->ws.bytes;
  char* h1 = (char*)ly->hcat.p;
  char *h2 = h1 + (int64_t)rows * d * es, *hc = h2 + (int64_t)rows * d * es;
  const LayeredLayer* prev = nullptr;   // the layer whose expert outputs wait in ly->y
  for (auto& L : ly->L) {
    const LayeredLayer& src = L.Nkv ? L : ly->L[L.d.kv_from];
    const int KB = (d + 31) / 32, Nqkv = L.Nq + L.Nkv;
    const bool ff = L.d.experts > 0;
    BlockNormArgs a{};
    a.x = g->x; a.d = d; a.groups = ly->c.norm_groups; a.eps = ly->c.eps;
    a.w1 = L.norm1; a.h1 = h1; a.out_scale = 1.0f;
    if (ff) {
      a.w2 = L.norm2; a.h2 = h2; a.h2_sorted = ly->hs.p; a.next_pos = route_of(L).pos; a.next_top = L.d.top;
    }
    gated_pending(ly, prev, use_state, a);
    a.write_x = 1;
    if (S == 1) {
      a.conv_w = L.conv_w; a.conv_ring = L.ring; a.hc = hc; a.taps = ly->c.conv_taps; a.T0 = T0; a.state = dT;
    }
    PROF(KC_NORM, launch_block_norm(dev, dt, a, rows, g->s));
    if (S > 1) PROF(KC_NORM, launch_short_conv(dev, g->st, dt, hc, h1, L.conv_w, L.ring, B, S, d, ly->c.conv_taps, T0, dT, g->gather_lens, g->s));
    // gates and projections
    {
      Epilogue e1 = make_ep(L.g1b, nullptr, ly->gate1.p, nullptr, TSB200_ACT_SIGMOID, 0);
      Epilogue e2 = make_ep(L.g2b, nullptr, ly->gate2.p, nullptr, TSB200_ACT_SIGMOID, 0);
      Epilogue e3 = make_ep(nullptr, nullptr, ly->qkv.p, nullptr, TSB200_ACT_NONE, 0);
      int r = 2;
      if (rows <= 64 && ff) {
        const LinearSection sec[3] = {{d, e1, 0}, {d, e2, 1}, {Nqkv, e3, 2}};
        prof_begin(g, KC_LINEAR);
        r = launch_gemm_stream_sections(dev, g->st, dt, h1, L.fused, rows, d, sec, 3, pdl, ws, wsb, g->s);
        if (r == 0) return 0;
        if (r == 1) prof_end(g, KC_LINEAR);
      }
      if (r == 2) {
        PROF(KC_LINEAR, launch_linear(dev, g->st, dt, h1, L.fused, rows, d, d, e1, ws, wsb, g->s, true));
        if (ff) PROF(KC_LINEAR, launch_linear(dev, g->st, dt, h2, (char*)L.fused + (int64_t)L.ct_gate2 * KB * 16384, rows, d, d, e2, ws, wsb, g->s, true));
        PROF(KC_LINEAR, launch_linear(dev, g->st, dt, hc, (char*)L.fused + (int64_t)L.ct_qkv * KB * 16384, rows, d, Nqkv, e3, ws, wsb, g->s, true));
      }
    }
    const int64_t seq_stride = (int64_t)g->c.max_tokens * src.sh.row;
    LatentArgs at{};
    at.shape = L.sh; at.q = ly->qkv.p; at.q_stride = Nqkv; at.dkv_col = L.Nkv ? L.Nq : -1; at.norm_w = L.kv_norm; at.eps = ly->c.eps; at.tab = L.tab;
    at.cache = src.cache; at.seq_stride = seq_stride;
    at.B = B; at.S = S; at.T0 = T0; at.Tmax = g->c.max_tokens; at.state = dT;
    at.splits = latent_pick_splits(g->st, L.sh, B, S, T_plan);
    at.uk = L.uk; at.uv = L.uv; at.ukv_packed = L.ukv; at.q_lat = ly->q_lat.p; at.part = (float*)ly->part.p; at.part_elems = ly->part.bytes / 4;
    at.kv = ly->kv.p; at.kv_elems = ly->kv.bytes / es; at.compact = ly->compact.p; at.compact_elems = ly->compact.bytes / es; at.out = ly->attn.p; at.lin_ws = ws; at.lin_ws_bytes = wsb;
    PROF(KC_ATTENTION, launch_latent_attention(dev, g->st, dt, at, g->s));
    {
      Epilogue e = make_ep(nullptr, g->x, nullptr, g->x, TSB200_ACT_NONE, 0);
      e.gate = ly->gate1.p;
      PROF(KC_LINEAR, launch_linear(dev, g->st, dt, ly->attn.p, L.wo, rows, L.sh.H * L.sh.vdim, d, e, ws, wsb, g->s, true));
    }
    prev = nullptr;
    if (ff) {
      const int picks = rows * L.d.top;
      RowGroups gr{};
      gr.table = route_of(L).blocks; gr.n_blocks = route_of(L).n_blocks;
      gr.max_blocks = layered_max_blocks(picks, L.d.experts, rt.block);
      auto grouped = [&](const void* x, const void* W, int64_t matrix_bytes, int K, int N, const Epilogue& e) -> int {
        gr.matrix_bytes = matrix_bytes;
        int r = 2;
        if (rt.block <= 16) r = launch_gemm_stream_grouped(dev, g->st, dt, x, W, picks, rt.block, K, N, e, gr, pdl, ws, wsb, g->s);
        if (r == 2) r = launch_gemm_tc_grouped(dev, g->st, dt, x, W, picks, K, N, e, gr, g->s);
        if (r == 2) r = launch_pick_linear(dev, dt, x, W, route_of(L).matrix_of, matrix_bytes, picks, K, N, e, g->s);
        return r;
      };
      Epilogue eu = make_ep(nullptr, nullptr, ly->hidden.p, nullptr, TSB200_ACT_CLAMP_GLU, 1);
      eu.glu_limit = L.d.glu_limit; eu.glu_slope = L.d.glu_slope; eu.glu_shift = L.d.glu_shift;
      PROF(KC_EXPERTS, grouped(ly->hs.p, L.up, L.up_bytes, d, 2 * L.d.ff, eu));
      PROF(KC_EXPERTS, grouped(ly->hidden.p, L.down, L.down_bytes, L.d.ff, d, make_ep(nullptr, nullptr, ly->y.p, nullptr, TSB200_ACT_NONE, 0)));
      prev = &L;
    }
  }
  ps.last = prev;
  return 1;
}

// A sublayer's output that joins the residual in the next sandwich norm.
static void sandwich_pending(const Layered* ly, const LayeredLayer* prev, SandwichNormArgs& a) {
  if (!prev) return;
  a.y = ly->y.p;
  a.post_w = prev->d.ff > 0 ? prev->norm2b : prev->norm1b;
  a.scale = prev->d.ff > 0 ? prev->scale2 : prev->scale1;
}

// Layers of sandwich blocks; the last sublayer's output stays pending.
static int sandwich_layers(Gpt* g, LayerPass& ps) {
  Layered* ly = g->ly;
  const int B = ps.B, S = ps.S;
  const int dev = g->c.device, dt = g->c.dtype, d = ly->c.d, rows = B * S;
  const int* dT = ps.use_state ? g->state : nullptr;
  void *h = ly->hcat.p, *ws = ly->ws.p;
  const int64_t wsb = ly->ws.bytes;
  const int NT = packed_tile_cols(dt);
  const LayeredLayer* prev = nullptr;
  auto linear = [&](const void* x, const void* W, int K, int N, const Epilogue& e) { return launch_linear(dev, g->st, dt, x, W, rows, K, N, e, ws, wsb, g->s, true); };
  for (auto& L : ly->L) {
    SandwichNormArgs a{};
    a.x = g->x; a.d = d; a.eps = ly->c.eps; a.write_x = 1; a.h = h;
    a.next_w = L.norm1;
    sandwich_pending(ly, prev, a);
    PROF(KC_NORM, launch_sandwich_norm(dev, dt, a, rows, g->s));
    const Epilogue eq = make_ep(L.qkv_b, nullptr, ly->qkv.p, nullptr, TSB200_ACT_NONE, 0);
    if (L.d.mixer == TSB200_MIXER_GROUPED) {
      PROF(KC_LINEAR, linear(h, L.fused, d, L.Nq, eq));
      const LayeredLayer& src = L.d.kv_from < 0 ? L : ly->L[L.d.kv_from];
      GroupedArgs at{};
      at.shape = L.gs; at.qkv = ly->qkv.p; at.q_stride = L.Nq; at.k_col = L.k_col; at.v_col = L.v_col; at.g_col = L.g_col;
      at.q_norm = L.q_norm; at.k_norm = L.k_norm; at.bias = L.bias; at.sink = L.sink; at.cK = src.cK; at.cV = src.cV;
      at.B = B; at.S = S; at.T0 = ps.T0; at.Tmax = g->c.max_tokens; at.state = dT;
      at.splits = S == 1 ? grouped_pick_splits(g->st, dt, L.gs, B, ps.T_plan) : 1;
      at.qn = ly->q_lat.p; at.part = (float*)ly->part.p; at.part_elems = ly->part.bytes / 4; at.counters = (unsigned int*)ly->counters.p; at.out = ly->attn.p;
      PROF(KC_ATTENTION, launch_grouped_attention(dev, g->st, dt, at, g->s));
    } else {
      // the gates' logits stay fp32: a section of their own on the same rows
      const Epilogue eg = make_ep(L.gates_b, nullptr, nullptr, (float*)ly->gates.p, TSB200_ACT_NONE, 0);
      const LinearSection sec[2] = {{L.Nq, eq, 0}, {2 * L.ms.H, eg, 0}};
      prof_begin(g, KC_LINEAR);
      const int r = launch_gemm_stream_sections(dev, g->st, dt, h, L.fused, rows, d, sec, 2, g->pdl, ws, wsb, g->s);
      if (r == 0) return 0;
      if (r == 1) prof_end(g, KC_LINEAR);
      if (r == 2) {
        const int64_t tile = (int64_t)((d + 31) / 32) * 32 * NT * g->es;
        PROF(KC_LINEAR, linear(h, L.fused, d, L.Nq, eq));
        PROF(KC_LINEAR, linear(h, (char*)L.fused + L.ct_gates * tile, d, 2 * L.ms.H, eg));
      }
      MemoryArgs m{};
      m.shape = L.ms; m.x = ly->qkv.p; m.stride = L.Nq; m.gates = (const float*)ly->gates.p; m.norm_w = L.mem_norm; m.state = (float*)L.mem;
      m.B = B; m.S = S; m.T0 = ps.T0; m.step_state = dT; m.lens = g->gather_lens; m.ids = g->ids_cur; m.stop_fin = ps.use_state ? g->stop_fin : 0;
      m.scratch = ly->chunks.p; m.scratch_bytes = ly->chunks.bytes; m.out = ly->attn.p;
      PROF(KC_MEMORY, launch_matrix_memory(dev, g->st, dt, m, g->s));
    }
    PROF(KC_LINEAR, linear(ly->attn.p, L.wo, L.mixed_cols(), d, make_ep(nullptr, nullptr, ly->y.p, nullptr, TSB200_ACT_NONE, 0)));
    if (L.d.ff > 0) {
      a.y = ly->y.p; a.post_w = L.norm1b; a.scale = L.scale1; a.next_w = L.norm2;
      PROF(KC_NORM, launch_sandwich_norm(dev, dt, a, rows, g->s));
      PROF(KC_LINEAR, linear(h, L.up, d, 2 * L.d.ff, make_ep(nullptr, nullptr, ly->hidden.p, nullptr, TSB200_ACT_SILU, 1)));
      PROF(KC_LINEAR, linear(ly->hidden.p, L.down, L.d.ff, d, make_ep(nullptr, nullptr, ly->y.p, nullptr, TSB200_ACT_NONE, 0)));
    }
    prev = &L;
  }
  ps.last = prev;
  return 1;
}

// Forward pass over B * S new tokens (ids in g->ids_in, or g->ids_cur in a captured step); logits of each sequence's last position
// to g->logits, or of the rows g->want_rows (device, g->n_want of them) to g->want_logits.  T_plan: the longest cache the splits of
// the attention are chosen for.
static int enqueue_layered(Gpt* g, int B, int S, int T0, bool use_state, int T_plan) {
  NvtxRange nvtx_(S == 1 ? "tsb200.forward.step" : "tsb200.forward.prompt");
  // sandwich blocks, ms per step with / without chained launches: 8 sequences 1.07 / 1.10 (4k), 16: 1.29 / 1.30, 32: 1.06 / 1.03 (2k), 64: 1.56 / 1.43
  PdlScope pdl_scope(g->pdl && S == 1 && (B <= 16 || g->ly->c.block != TSB200_BLOCK_SANDWICH));
  Layered* ly = g->ly;
  const int dev = g->c.device, dt = g->c.dtype, d = ly->c.d, rows = B * S;
  const int* dT = use_state ? g->state : nullptr;
  TSB_CHECK(ly->missing.empty(), "layered engine: %d weights have not been given, the first is '%s'", (int)ly->missing.size(), ly->missing.begin()->c_str());
  const int* ids = (S == 1 && use_state) ? g->ids_cur : g->ids_in;
  const bool sandwich = ly->c.block == TSB200_BLOCK_SANDWICH;
  const Layered::Routing& rt = ly->routing[use_state ? 1 : 0];
  void *ws = ly->ws.p;
  const int64_t wsb = ly->ws.bytes;
  g->lin_syms_used = true;
  {
    prof_begin(g, KC_EMBED);
    const int gsz = rows < g->st->sm_count * 8 ? rows : g->st->sm_count * 8;
    if (dt == TSB200_F32)
      TSB_CUDA(launch_k(embed_kernel<float>, dim3(gsz), dim3(256), 0, g->s, g->x, (const float*)g->E, (const float*)nullptr, ids, rows, S, d, g->c.V, ly->c.embed_scale, 0, 0, T0, dT));
    else
      TSB_CUDA(launch_k(embed_kernel<__nv_bfloat16>, dim3(gsz), dim3(256), 0, g->s, g->x, (const __nv_bfloat16*)g->E, (const __nv_bfloat16*)nullptr, ids, rows, S, d, g->c.V, ly->c.embed_scale, 0, 0, T0, dT));
    count_launch(dev);
    TSB_TRY(check_launch("embed"));
    TSB_TRY(launch_table_route(dev, (const RouteLayer*)rt.layers.p, ly->n_route, ly->max_experts, ids, rows, g->c.V, rt.block, g->s));
    prof_end(g, KC_EMBED);
  }
  LayerPass ps{B, S, T0, T_plan, use_state, nullptr};
  TSB_TRY(sandwich ? sandwich_layers(g, ps) : gated_layers(g, ps));
  // final norm on the rows whose logits are asked for, head
  const int n_out = g->want_rows ? g->n_want : B;
  if (n_out == 0) return 1;
  void* hl = g->want_rows ? g->want_h : g->hl;
  if (sandwich) {
    SandwichNormArgs a{};
    a.x = g->x; a.d = d; a.eps = ly->c.eps; a.next_w = g->nf_g; a.h = hl;
    sandwich_pending(ly, ps.last, a);
    a.rows_of = g->want_rows;
    if (!g->want_rows && S > 1) { a.last_of_S = S; a.lens = g->gather_lens; }
    PROF(KC_NORM, launch_sandwich_norm(dev, dt, a, n_out, g->s));
  } else {
    BlockNormArgs a{};
    a.x = g->x; a.d = d; a.groups = ly->c.norm_groups; a.eps = ly->c.eps; a.w1 = g->nf_g; a.h1 = hl; a.out_scale = ly->c.logit_scale;
    gated_pending(ly, ps.last, use_state, a);
    a.rows_of = g->want_rows;
    if (!g->want_rows && S > 1) { a.last_of_S = S; a.lens = g->gather_lens; }
    PROF(KC_NORM, launch_block_norm(dev, dt, a, n_out, g->s));
  }
  PROF(KC_LINEAR, launch_linear(dev, g->st, dt, hl, g->head_w, n_out, d, g->c.V, make_ep(nullptr, nullptr, nullptr, g->want_rows ? g->want_logits : g->logits, TSB200_ACT_NONE, 0),
                                ws, wsb, g->s, true));
  return 1;
}

// bytes a decode step of B sequences at cache length T has to move: weights once (experts: as many as B tokens can name), the
// cache rows every layer reads and writes, convolution states, logits
static int64_t layered_step_bytes(const Gpt* g, int B, int T) {
  const Layered* ly = g->ly;
  const int64_t d = ly->c.d, es = g->es;
  int64_t n = d * ly->c.V + d;
  int64_t total = 0;
  for (auto& L : ly->L) {
    if (ly->c.block == TSB200_BLOCK_SANDWICH) {
      n += d * L.Nq + (int64_t)L.mixed_cols() * d + 3 * d * L.d.ff + (L.d.ff > 0 ? 6 : 3) * d;
      if (L.d.mixer == TSB200_MIXER_GROUPED) {
        const int64_t seen = L.gs.window > 0 ? std::min<int64_t>(T, L.gs.window + L.gs.keep_first) : T;
        total += (int64_t)B * L.gs.G * (L.gs.dim + L.gs.vdim) * es * (seen + (L.d.kv_from < 0 ? 1 : 0));
      } else {
        n += 2 * d * L.ms.H;
        total += 2 * (int64_t)B * memory_state_floats(L.ms) * 4;
      }
      continue;
    }
    const int64_t ex = std::min<int64_t>(L.d.experts, (int64_t)B * std::max(L.d.top, 0));
    n += (L.d.experts > 0 ? 2 : 1) * d * d + d * (L.Nq + L.Nkv) + (int64_t)L.sh.H * (L.sh.dim + L.sh.vdim) * L.sh.rank + (int64_t)L.sh.H * L.sh.vdim * d +
         3 * ex * d * L.d.ff + 4 * d + d * ly->c.conv_taps;
    total += (int64_t)B * T * (L.sh.rank + L.sh.rot) * es + (L.Nkv ? (int64_t)B * L.Nkv * es : 0) + (int64_t)B * ly->c.conv_taps * d * es;
  }
  return total + n * es + (int64_t)B * d * es + (int64_t)B * ly->c.V * 4;
}

}  // namespace tsb
