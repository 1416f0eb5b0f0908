// Layered models (rewb200_model_create_layers): weights, caches and the forward of decoders whose layers are described
// one by one.  They share the engine's sessions, lanes, page pool, captured decode step, sampler and lm_head
// (engine.cu); this file has what differs per layer.
//
// A block is the parallel x += mixer(norm1(x)) + ff(norm2(x)), where one launch (residual_norm) adds both branches' f32
// slabs to the residual, adds what a loop adds ahead of a pass, and leaves both norms of the next layer run, and in small
// steps the feed-forward branch runs on the slot's second stream beside the mixer; or x += norm1(mixer(x)), then
// x += norm2(ff(x)), where one launch (output_norm) per sublayer sums its slabs, norms the sum and adds it; or the parallel
// block with one norm that both branches read.
//
// Device layouts beyond engine.cu's: rows and Linear outputs are padded to multiples of 8 elements (zero weights, zero
// norm weights), so any width can be loaded by TMA; a mixer's input projections are one matrix; the key and value
// projections of a latent are one matrix; a loop's passes share weights and have a cache each.
#include <cmath>
#include <map>

#include "engine.cuh"

namespace rewb {

namespace {

int64_t pad8(int64_t v) { return (v + 7) / 8 * 8; }

enum Slot : int {
  SL_NORM1, SL_DQ, SL_DQ_NORM, SL_UQ, SL_DKV, SL_DKV_NORM, SL_UK, SL_UV, SL_G, SL_O, SL_NORM2, SL_GATE, SL_UP, SL_DOWN, SL_ROUTER,
  SL_E_GATE, SL_E_UP, SL_E_DOWN, SL_EMBED, SL_STEP, SL_FINAL, SL_HEAD, SL_Q, SL_K, SL_V, SL_Q_NORM, SL_K_NORM, SL_REL, SL_SINK, SL_A1, SL_A2,
  SL_A2_B, SL_V_GATE, SL_V_NORM, SL_ROUTER_B, SL_S_GATE, SL_S_UP, SL_S_DOWN, SL_Q_CONV, SL_K_CONV, SL_S_SG
};
enum Block : int { BLOCK_PARALLEL = 0, BLOCK_OUTPUT_NORM = 1, BLOCK_ONE_NORM = 2 };
enum Sink : int { SINK_NONE = 0, SINK_LEARNED = 1, SINK_ONE = 2 };
enum Mixer : int { MIX_LATENT = 1, MIX_GQA = 2, MIX_GLA = 3 };
struct TensorAt {
  Slot slot;
  int layer, expert;
};

// The canonical tensors of a layered model (rew_b200/layered.py lists the same).
void tensors_of(const rewb200_model* m, std::vector<TensorAt>* out) {
  out->push_back({SL_EMBED, -1, -1});
  if (m->stack.loop_times > 0) out->push_back({SL_STEP, -1, -1});
  for (int l = 0; l < m->cfg.n_layers; ++l) {
    const rewb200_layer& L = m->spec[l];
    auto add = [&](std::initializer_list<Slot> slots) {
      for (Slot s : slots) out->push_back({s, l, -1});
    };
    add({SL_NORM1});
    const bool own = L.kv_from < 0;
    if (L.mixer == MIX_LATENT) {
      add({SL_DQ, SL_DQ_NORM, SL_UQ});
      if (own) add({SL_DKV, SL_DKV_NORM});
      add({SL_UK, SL_UV});
      if (L.sink == SINK_LEARNED) add({SL_SINK});
    }
    if (L.mixer == MIX_GQA) {
      add({SL_Q});
      if (own) add({SL_K});
      if (own && !L.values_from_keys) add({SL_V});
      if (L.conv_taps > 0) add({SL_Q_CONV});
      if (L.conv_taps > 0 && own) add({SL_K_CONV});
      if (L.qk_norm) add({SL_Q_NORM});
      if (L.qk_norm && own) add({SL_K_NORM});
      if (L.bias_rows > 0) add({SL_REL});
      if (L.sink == SINK_LEARNED) add({SL_SINK});
    }
    if (L.mixer == MIX_GLA) add({SL_Q, SL_K, SL_V, SL_A1, SL_A2, SL_A2_B, SL_V_GATE, SL_V_NORM});
    if (L.out_gate) out->push_back({SL_G, l, -1});
    out->push_back({SL_O, l, -1});
    if (L.ff && m->stack.block != BLOCK_ONE_NORM) out->push_back({SL_NORM2, l, -1});
    if (L.ff == 1)
      for (Slot s : {SL_GATE, SL_UP, SL_DOWN}) out->push_back({s, l, -1});
    if (L.ff == 2) {
      add({SL_ROUTER});
      if (L.router_bias) add({SL_ROUTER_B});
      for (int e = 0; e < L.experts; ++e) {
        if (L.expert_gated) out->push_back({SL_E_GATE, l, e});
        out->push_back({SL_E_UP, l, e});
        out->push_back({SL_E_DOWN, l, e});
      }
      if (L.shared_ffn > 0) add({SL_S_GATE, SL_S_UP, SL_S_DOWN});
      if (L.shared_gate) add({SL_S_SG});
    }
  }
  out->push_back({SL_FINAL, -1, -1});
  if (m->stack.own_head) out->push_back({SL_HEAD, -1, -1});
}

int shape_of(const rewb200_model* m, const TensorAt& t, int64_t* rows, int64_t* cols, bool* vec) {
  const int64_t d = m->cfg.d_model;
  const rewb200_layer* L = t.layer >= 0 ? &m->spec[t.layer] : nullptr;
  *vec = false;
  auto mat = [&](int64_t r, int64_t c) { *rows = r; *cols = c; };
  auto v = [&](int64_t n) { *rows = 1; *cols = n; *vec = true; };
  switch (t.slot) {
    case SL_EMBED: mat(m->cfg.vocab, d); break;
    case SL_STEP: mat(m->stack.loop_times, d); break;
    case SL_FINAL: case SL_NORM1: case SL_NORM2: v(d); break;
    case SL_DQ: mat(d, L->q_rank); break;
    case SL_DQ_NORM: v(L->q_rank); break;
    case SL_UQ: mat(L->q_rank, (int64_t)L->heads * (L->dim + L->rot_dim)); break;
    case SL_DKV: mat(d, L->kv_rank + L->rot_dim); break;
    case SL_DKV_NORM: v(L->kv_rank); break;
    case SL_UK: mat(L->kv_rank, (int64_t)L->heads * L->dim); break;
    case SL_UV: mat(L->kv_rank, (int64_t)L->heads * L->vdim); break;
    case SL_G: mat(d, L->heads); break;
    case SL_O: mat((int64_t)L->heads * L->vdim, d); break;
    case SL_GATE: case SL_UP: case SL_E_GATE: case SL_E_UP: mat(d, L->ffn); break;
    case SL_DOWN: case SL_E_DOWN: mat(L->ffn, d); break;
    case SL_ROUTER: mat(d, L->experts); break;
    case SL_ROUTER_B: v(L->experts); break;
    case SL_S_GATE: case SL_S_UP: mat(d, L->shared_ffn); break;
    case SL_S_DOWN: mat(L->shared_ffn, d); break;
    case SL_HEAD: mat(d, m->cfg.vocab); break;
    case SL_Q: mat(d, (int64_t)L->heads * L->dim); break;
    case SL_K: mat(d, (int64_t)(L->mixer == MIX_GQA ? L->kv_heads : L->heads) * L->dim); break;
    case SL_V: mat(d, (int64_t)(L->mixer == MIX_GQA ? L->kv_heads : L->heads) * L->vdim); break;
    case SL_Q_NORM: case SL_K_NORM: v(L->dim); break;
    case SL_REL: mat(L->bias_rows, L->heads); break;
    case SL_SINK: v(L->heads); break;
    case SL_A1: mat(d, L->decay_rank); break;
    case SL_A2: mat(L->decay_rank, (int64_t)L->heads * L->dim); break;
    case SL_A2_B: v((int64_t)L->heads * L->dim); break;
    case SL_V_GATE: mat(d, (int64_t)L->heads * L->vdim); break;
    case SL_V_NORM: v(L->vdim); break;
    case SL_Q_CONV: mat((int64_t)L->heads * L->dim, L->conv_taps); break;
    case SL_K_CONV: mat((int64_t)L->kv_heads * L->dim, L->conv_taps); break;
    case SL_S_SG: mat(d, 1); break;
  }
  return REWB200_OK;
}

int locate_tensor(const rewb200_model* m, int64_t index, TensorAt* out) {
  std::vector<TensorAt> all;
  tensors_of(m, &all);
  RB_REQUIRE(index >= 0 && index < (int64_t)all.size(), "tensor index " + std::to_string(index) + " out of range");
  *out = all[index];
  return REWB200_OK;
}

__global__ void add_scalar_kernel(float* p, int64_t n, float v) {
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) p[i] += v;
}
// dst[c][r] = src[r][c] for a [rows, cols] matrix (model dtype on both sides), row strides lds / ldd
template <typename T>
__global__ void transpose_kernel(const T* src, int64_t lds, T* dst, int64_t ldd, int64_t rows, int64_t cols) {
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= rows * cols) return;
  const int64_t c = i / rows, r = i % rows;
  dst[c * ldd + r] = src[r * lds + c];
}

int zero_weights(rewb200_model* m, void** p, size_t bytes) {
  RB_TRY(dev_alloc(m, p, bytes));
  RB_CUDA(cudaMemsetAsync(*p, 0, std::max<size_t>(bytes, 256), m->c->stream));
  return REWB200_OK;
}
int zero_lin(rewb200_model* m, LinW* w, int64_t K, int64_t N) {
  RB_TRY(alloc_lin(m, w, K, N));
  RB_CUDA(cudaMemsetAsync(w->w, 0, (size_t)K * N * dtype_size(m->cfg.dtype), m->c->stream));
  return REWB200_OK;
}

// (cos, sin) of pos * base^(-2 i / dims), angles in double: the table is exact to f32 rounding at any position
int rope_table(rewb200_model* m, double base, int dims, float2** out) {
  std::vector<float2> t((size_t)m->cfg.max_seq * (dims / 2));
  for (int i = 0; i < dims / 2; ++i) {
    const double f = std::pow(base, -2.0 * i / dims);
    for (int p = 0; p < m->cfg.max_seq; ++p)
      t[(size_t)p * (dims / 2) + i] = make_float2((float)std::cos(p * f), (float)std::sin(p * f));
  }
  RB_TRY(dev_alloc(m, (void**)out, t.size() * sizeof(float2)));
  if (!t.empty()) RB_CUDA(cudaMemcpyAsync(*out, t.data(), t.size() * sizeof(float2), cudaMemcpyHostToDevice, m->c->stream));
  RB_CUDA(cudaStreamSynchronize(m->c->stream));
  return REWB200_OK;
}

// Row of a bias table of B rows for a key n tokens back: a row per distance below B / 2, then logarithmic ones up to D.
// The small allowance keeps distances that lie exactly on a border on its far side.
int distance_bucket(int n, int B, int D) {
  const int h = B / 2;
  if (n < h) return n;
  if (h == 0 || D <= h) return B - 1;
  const double v = std::log((double)n / h) / std::log((double)D / h) * (B - h);
  return (int)std::min<double>(B - 1, h + std::floor(v + 1e-9));
}
// Distances a bias table tells apart: 0 .. bias_distances - 1, the last one standing for all longer ones.
int bias_distances(int B, int D) {
  int n = 0;
  while (distance_bucket(n, B, D) < B - 1) ++n;
  return n + 1;
}

// Tables of a mixer-2 layer by distance: [heads][n_bias] from the stored [rows][heads].
int upload_bias(rewb200_model* m, const rewb200_layer& L, GqaDev& G, const float* host) {
  std::vector<float> t((size_t)L.heads * G.m.n_bias);
  for (int n = 0; n < G.m.n_bias; ++n) {
    const int b = distance_bucket(n, L.bias_rows, L.bias_max);
    for (int h = 0; h < L.heads; ++h) t[(size_t)h * G.m.n_bias + n] = host[(size_t)b * L.heads + h];
  }
  RB_CUDA(cudaMemcpyAsync(G.bias, t.data(), t.size() * sizeof(float), cudaMemcpyHostToDevice, m->c->stream));
  RB_CUDA(cudaStreamSynchronize(m->c->stream));
  return REWB200_OK;
}

// Convolution weights [taps][channels] from the stored [channels][taps] of queries or keys, whose first channel is c0.
int upload_conv(rewb200_model* m, const GqaDev& G, int64_t c0, int64_t channels, const float* host) {
  std::vector<float> t((size_t)G.m.taps * channels);
  for (int64_t ch = 0; ch < channels; ++ch)
    for (int j = 0; j < G.m.taps; ++j) t[(size_t)j * channels + ch] = host[ch * G.m.taps + j];
  RB_CUDA(cudaMemcpy2DAsync(G.conv + c0, gqa_channels(G.m) * sizeof(float), t.data(), channels * sizeof(float), channels * sizeof(float), G.m.taps,
                            cudaMemcpyHostToDevice, m->c->stream));
  RB_CUDA(cudaStreamSynchronize(m->c->stream));
  return REWB200_OK;
}

// The Linear weights of a layer's mixer that are no routed experts (all of them padded matrices of the model dtype).
std::vector<LinW*> mixer_linears(LayerDev& D) {
  if (D.mixer == MIX_LATENT) return {&D.a.in, &D.a.uq, &D.a.ukv, &D.o};
  if (D.mixer == MIX_GQA) return {&D.g.in, &D.o};
  return {&D.l.in, &D.o};
}
bool has_dense(const LayerDev& D) { return D.ffn_local > 0; }

}  // namespace

int layered_create(rewb200_model* m, const rewb200_layer* layers, const rewb200_stack* stack) {
  const int n = m->cfg.n_layers;
  const size_t es = dtype_size(m->cfg.dtype);
  m->layered = true;
  m->spec.assign(layers, layers + n);
  m->stack = *stack;
  const rewb200_stack& st = m->stack;
  RB_REQUIRE(st.loop_times >= 0 && (st.loop_times == 0 || (st.loop_start >= 0 && st.loop_start < st.loop_stop && st.loop_stop <= n)),
             "layered model: the loop must cover layers start .. stop - 1 of the stack");
  RB_REQUIRE(st.block >= BLOCK_PARALLEL && st.block <= BLOCK_ONE_NORM, "layered model: unknown block");
  RB_REQUIRE(st.block != BLOCK_OUTPUT_NORM || st.loop_times == 0, "layered model: blocks normed on the way back run without a loop");
  RB_REQUIRE(st.logit_softcap >= 0.f, "layered model: the cap of the logits must not be negative");
  for (int l = 0; l < n; ++l) {
    const rewb200_layer& L = m->spec[l];
    const std::string who = "layer " + std::to_string(l) + ": ";
    RB_REQUIRE(L.mixer >= MIX_LATENT && L.mixer <= MIX_GLA, who + "unknown mixer");
    RB_REQUIRE(L.heads > 0 && L.dim > 0 && L.vdim > 0, who + "mixer sizes must be positive");
    RB_REQUIRE(L.sink >= SINK_NONE && L.sink <= SINK_ONE, who + "unknown sink");
    RB_REQUIRE(L.conv_taps >= 0 && (L.mixer == MIX_GQA || (L.conv_taps == 0 && !L.values_from_keys)), who + "convolutions and values from keys belong to grouped-query attention");
    if (L.kv_from >= 0) {
      RB_REQUIRE(L.mixer != MIX_GLA && L.kv_from < l, who + "kv_from must name an earlier layer");
      const rewb200_layer& S = m->spec[L.kv_from];
      const bool same = L.mixer == MIX_LATENT ? S.kv_rank == L.kv_rank && S.rot_dim == L.rot_dim : S.kv_heads == L.kv_heads && S.dim == L.dim && S.vdim == L.vdim;
      RB_REQUIRE(S.mixer == L.mixer && S.kv_from < 0 && same, who + "kv_from must name a layer of the same mixer with latents, or keys and values, of its own and the same sizes");
    }
    if (L.mixer == MIX_LATENT) {
      RB_REQUIRE(L.rot_dim >= 0 && L.q_rank > 0 && L.kv_rank > 0, who + "mixer sizes must be positive");
      RB_REQUIRE(L.rope_dims >= 0 && L.rope_dims % 2 == 0 && L.rope_dims <= L.rot_dim, who + "rotated features must be pairs within rot_dim");
      RB_REQUIRE(L.window >= 0, who + "the window must not be negative");
    } else if (L.mixer == MIX_GQA) {
      RB_REQUIRE(L.kv_heads > 0 && L.heads % L.kv_heads == 0, who + "heads must be divisible by kv_heads");
      RB_REQUIRE(L.bias_rows >= 0 && (L.bias_rows == 0 || (L.bias_max > 0 && L.bias_max <= 1 << 20)), who + "the distance bias needs a positive bias_max");
      RB_REQUIRE(L.temp_every >= 0, who + "temp_every must not be negative");
      RB_REQUIRE(L.rope_dims >= 0 && L.rope_dims % 2 == 0 && L.rope_dims <= L.dim, who + "rotated features must be pairs within the head");
      RB_REQUIRE(!L.values_from_keys || L.vdim == L.dim, who + "values that are the keys have their size");
    } else {
      RB_REQUIRE(L.decay_rank > 0 && L.tau > 0.f, who + "decay_rank and tau must be positive");
    }
    RB_REQUIRE(L.ff >= 0 && L.ff <= 2 && (L.ff == 0 || L.ffn > 0), who + "unknown feed-forward");
    RB_REQUIRE(L.shared_ffn >= 0 && (L.ff == 2 || L.shared_ffn == 0), who + "a shared expert stands beside routed ones");
    RB_REQUIRE(!L.shared_gate || (L.shared_ffn > 0 && st.block != BLOCK_OUTPUT_NORM), who + "the gate of a shared expert needs one, in a parallel block");
    RB_REQUIRE(L.ff != 2 || (L.experts > 0 && L.experts <= 256 && L.top_k > 0 && L.top_k <= L.experts),
               who + "experts must be in 1..256 and top in 1..experts");
  }
  const int64_t d = m->cfg.d_model, dp = m->dp = pad8(d);
  m->vp = pad8(m->cfg.vocab);
  RB_TRY(zero_weights(m, &m->embed, (size_t)m->cfg.vocab * dp * es));
  if (st.loop_times > 0) RB_TRY(zero_weights(m, (void**)&m->step_vec, (size_t)st.loop_times * dp * sizeof(float)));
  std::map<std::pair<double, int>, float2*> tables;
  auto rope_of = [&](const rewb200_layer& L, const float2** out) -> int {
    if (L.rope_dims == 0) return REWB200_OK;
    float2*& t = tables[{L.rope_base, L.rope_dims}];
    if (!t) RB_TRY(rope_table(m, L.rope_base, L.rope_dims, &t));
    *out = t;
    return REWB200_OK;
  };
  // a sink of one is a score of zero: the zeros the array starts with
  auto sink_of = [&](const rewb200_layer& L, float** out) { return L.sink ? zero_weights(m, (void**)out, L.heads * sizeof(float)) : REWB200_OK; };
  m->layers.resize(n);
  int64_t widest = dp, q_cols = 0, attn_cols = 0;
  for (int l = 0; l < n; ++l) {
    const rewb200_layer& L = m->spec[l];
    LayerDev& D = m->layers[l];
    D.mixer = L.mixer;
    RB_TRY(zero_weights(m, (void**)&D.ln1g, dp * sizeof(float)));
    if (L.ff && st.block != BLOCK_ONE_NORM) RB_TRY(zero_weights(m, (void**)&D.ln2g, dp * sizeof(float)));
    const bool own = L.kv_from < 0;
    if (L.mixer == MIX_LATENT) {
      LatentDev& A = D.a;
      A.m = LatentDims{L.heads, L.dim, L.rot_dim, L.vdim, L.q_rank, L.kv_rank, L.rope_dims, L.window, L.out_gate, L.scale, nullptr, m->cfg.max_seq, own ? 1 : 0, nullptr};
      RB_TRY(rope_of(L, &A.m.rope));
      RB_TRY(sink_of(L, &A.sink));
      A.m.sink = A.sink;
      RB_TRY(zero_lin(m, &A.in, dp, pad8((int64_t)L.q_rank + (own ? L.kv_rank + L.rot_dim : 0) + (L.out_gate ? L.heads : 0))));
      RB_TRY(zero_lin(m, &A.uq, pad8(L.q_rank), pad8((int64_t)L.heads * (L.dim + L.rot_dim))));
      RB_TRY(zero_lin(m, &A.ukv, L.kv_rank, pad8((int64_t)L.heads * (L.dim + L.vdim))));
      RB_TRY(zero_weights(m, (void**)&A.q_norm, L.q_rank * sizeof(float)));
      if (own) RB_TRY(zero_weights(m, (void**)&A.kv_norm, L.kv_rank * sizeof(float)));
      A.ldc = pad8(L.kv_rank + L.rot_dim);
      widest = std::max(widest, std::max(A.in.N, A.uq.N));
      q_cols = std::max(q_cols, A.uq.N);
    } else if (L.mixer == MIX_GQA) {
      GqaDev& G = D.g;
      G.ldk = pad8(L.dim);
      G.ldv = pad8(L.vdim);
      RB_TRY(zero_lin(m, &G.in, dp, pad8((int64_t)L.heads * L.dim + (own ? (int64_t)L.kv_heads * (L.dim + (L.values_from_keys ? 0 : L.vdim)) : 0) + (L.out_gate ? L.heads : 0))));
      if (L.qk_norm) RB_TRY(zero_weights(m, (void**)&G.q_norm, L.dim * sizeof(float)));
      if (L.qk_norm && own) RB_TRY(zero_weights(m, (void**)&G.k_norm, L.dim * sizeof(float)));
      const int nb = L.bias_rows > 0 ? bias_distances(L.bias_rows, L.bias_max) : 0;
      if (nb > 0) RB_TRY(zero_weights(m, (void**)&G.bias, (size_t)L.heads * nb * sizeof(float)));
      RB_TRY(sink_of(L, &G.sink));
      G.m = GqaDims{L.heads, L.kv_heads, L.dim, L.vdim, own ? 1 : 0, L.out_gate, L.scale, G.q_norm, G.k_norm, L.temp_every, L.temp_coef, G.bias, nb, G.sink,
                    L.values_from_keys, L.conv_taps, nullptr, L.rope_dims, nullptr};
      RB_TRY(rope_of(L, &G.m.rope));
      if (L.conv_taps > 0) RB_TRY(zero_weights(m, (void**)&G.conv, (size_t)L.conv_taps * gqa_channels(G.m) * sizeof(float)));
      G.m.conv = G.conv;
      widest = std::max(widest, G.in.N);
      q_cols = std::max(q_cols, pad8((int64_t)L.heads * L.dim));
    } else {
      GlaDev& A = D.l;
      const int64_t hk = (int64_t)L.heads * L.dim, hv = (int64_t)L.heads * L.vdim;
      RB_TRY(zero_lin(m, &A.in, dp, pad8(2 * hk + 2 * hv + L.decay_rank)));
      RB_TRY(zero_weights(m, (void**)&A.a2, hk * L.decay_rank * sizeof(float)));
      RB_TRY(zero_weights(m, (void**)&A.a2_b, hk * sizeof(float)));
      RB_TRY(zero_weights(m, (void**)&A.norm, L.vdim * sizeof(float)));
      A.m = GlaDims{L.heads, L.dim, L.vdim, L.decay_rank, L.tau, A.a2, A.a2_b, A.norm};
      widest = std::max(widest, A.in.N);
    }
    RB_TRY(zero_lin(m, &D.o, pad8((int64_t)L.heads * L.vdim), dp));
    attn_cols = std::max(attn_cols, D.o.K);
    D.ff = L.ff;
    const int64_t fp = pad8(L.ffn);
    if (L.ff == 1) {
      D.ffn_local = fp;
      m->max_ffn = std::max(m->max_ffn, fp);
      RB_TRY(zero_lin(m, &D.gu, dp, 2 * fp));
      RB_TRY(zero_lin(m, &D.down, fp, dp));
    } else if (L.ff == 2) {
      MoeDev& X = D.x;
      D.moe = true;
      X.E = X.E_l = L.experts;
      X.top_k = L.top_k;
      X.renorm = L.renormalize;
      X.scale = L.router_scale == 0.f ? 1.f : L.router_scale;
      X.shared_gate = L.shared_gate != 0;
      X.gated = L.expert_gated != 0;
      X.f = fp;
      const int64_t up = X.gated ? 2 * fp : fp;
      RB_TRY(zero_lin(m, &X.router, dp, pad8(L.experts + (X.shared_gate ? 1 : 0))));
      RB_TRY(zero_weights(m, &X.gu, (size_t)L.experts * dp * up * es));
      RB_TRY(zero_weights(m, &X.down, (size_t)L.experts * fp * dp * es));
      RB_TRY(zero_weights(m, (void**)&X.gu_b, (size_t)L.experts * up * sizeof(float)));
      RB_TRY(zero_weights(m, (void**)&X.down_b, (size_t)L.experts * dp * sizeof(float)));
      m->max_moe_ffn = std::max(m->max_moe_ffn, fp);
      m->max_experts = std::max<int>(m->max_experts, (int)X.router.N);
      m->max_topk = std::max(m->max_topk, X.top_k);
      if (L.shared_ffn > 0) {
        D.ffn_local = pad8(L.shared_ffn);
        m->max_ffn = std::max(m->max_ffn, D.ffn_local);
        RB_TRY(zero_lin(m, &D.gu, dp, 2 * D.ffn_local));
        RB_TRY(zero_lin(m, &D.down, D.ffn_local, dp));
      }
    }
  }
  m->nq = std::max(q_cols, attn_cols);  // sizes the query and attention-output buffers
  m->nqkv = widest;                     // ... and the split-K slabs
  RB_TRY(zero_weights(m, (void**)&m->ng, dp * sizeof(float)));
  RB_TRY(zero_lin(m, &m->lm, dp, m->vp));
  const int a = st.loop_times > 0 ? st.loop_start : n, b = st.loop_times > 0 ? st.loop_stop : n;
  for (int l = 0; l < a; ++l) m->runs.push_back({l, false, -1});
  for (int p = 0; p < st.loop_times; ++p)
    for (int l = a; l < b; ++l) m->runs.push_back({l, l == a && p > 0, l == a ? p : -1});
  for (int l = b; l < n; ++l) m->runs.push_back({l, false, -1});
  for (size_t r = 0; r < m->runs.size(); ++r) {
    LayerRun& R = m->runs[r];
    if (m->layers[R.layer].moe) ++m->n_moe;
    R.cache = (int)r;
    const rewb200_layer& L = m->spec[R.layer];
    if (L.mixer != MIX_GLA && L.kv_from >= 0)   // the latest run of that layer: in a loop, the one of the same pass
      for (size_t q = 0; q < r; ++q)
        if (m->runs[q].layer == L.kv_from) R.cache = (int)q;
  }
  RB_CUDA(cudaStreamSynchronize(m->c->stream));
  return REWB200_OK;
}

int64_t layered_tensor_count(const rewb200_model* m) {
  std::vector<TensorAt> all;
  tensors_of(m, &all);
  return (int64_t)all.size();
}

int layered_tensor_shape(const rewb200_model* m, int64_t index, int* ndims, int64_t* shape) {
  TensorAt t;
  RB_TRY(locate_tensor(m, index, &t));
  bool vec;
  int64_t r, c;
  RB_TRY(shape_of(m, t, &r, &c, &vec));
  *ndims = vec ? 1 : 2;
  shape[0] = vec ? c : r;
  shape[1] = vec ? 0 : c;
  return REWB200_OK;
}

int layered_set_tensor(rewb200_model* m, int64_t index, const float* host, int64_t numel) {
  TensorAt t;
  RB_TRY(locate_tensor(m, index, &t));
  bool vec;
  int64_t R, C;
  RB_TRY(shape_of(m, t, &R, &C, &vec));
  RB_REQUIRE(numel == R * C, "tensor " + std::to_string(index) + ": expected " + std::to_string(R * C) + " elements, got " + std::to_string(numel));
  RB_TRY(upload_stage(m, host, numel));
  const bool bf = m->cfg.dtype == REWB200_BF16;
  const size_t es = dtype_size(m->cfg.dtype);
  auto norm = [&](float* dst, bool zero_centred) -> int {
    RB_TRY(scatter(m, C, 0, 0, 1, C, dst, false, C, C, C, 0));
    if (zero_centred) {
      add_scalar_kernel<<<(unsigned)((C + 255) / 256), 256, 0, m->c->stream>>>(dst, C, 1.0f);
      RB_CUDA(cudaGetLastError());
    }
    return REWB200_OK;
  };
  auto cols = [&](void* w, int64_t ld, int64_t off) { return scatter(m, C, 0, 0, R, C, w, true, ld, C, C, off); };
  const bool zc = m->stack.norm_zero_centred != 0;
  if (t.slot == SL_EMBED) {
    RB_TRY(cols(m->embed, m->dp, 0));
    if (m->stack.own_head) return REWB200_OK;
    // the output head is the same table: the lm_head matrix is its transpose
    const int64_t n = R * C;
    if (bf)
      transpose_kernel<bf16><<<(unsigned)((n + 255) / 256), 256, 0, m->c->stream>>>((const bf16*)m->embed, m->dp, (bf16*)m->lm.w, m->vp, R, C);
    else
      transpose_kernel<float><<<(unsigned)((n + 255) / 256), 256, 0, m->c->stream>>>((const float*)m->embed, m->dp, (float*)m->lm.w, m->vp, R, C);
    RB_CUDA(cudaGetLastError());
    return REWB200_OK;
  }
  if (t.slot == SL_STEP) return scatter(m, C, 0, 0, R, C, m->step_vec, false, m->dp, C, C, 0);
  if (t.slot == SL_FINAL) return norm(m->ng, zc);
  if (t.slot == SL_HEAD) return cols(m->lm.w, m->vp, 0);
  LayerDev& D = m->layers[t.layer];
  const rewb200_layer& L = m->spec[t.layer];
  LatentDev& A = D.a;
  const int64_t fp = pad8(L.ffn);
  // gate / up columns of `f` logical ones: bf16 interleaves groups of 8, f32 concatenates
  auto gate_up = [&](void* w, bool up, int64_t f) {
    return scatter(m, C, 0, 0, R, C, w, true, 2 * pad8(f), bf ? 8 : f, bf ? 16 : f, up ? (bf ? 8 : pad8(f)) : 0);
  };
  auto vector = [&](float* dst) { return scatter(m, C, 0, 0, 1, R * C, dst, false, R * C, R * C, R * C, 0); };
  const int64_t hk = (int64_t)L.heads * L.dim, hv = (int64_t)L.heads * L.vdim;
  if (L.mixer == MIX_GQA) {
    GqaDev& G = D.g;
    const int64_t kv = L.kv_from < 0 ? (int64_t)L.kv_heads : 0;
    switch (t.slot) {
      case SL_Q: return cols(G.in.w, G.in.N, 0);
      case SL_K: return cols(G.in.w, G.in.N, hk);
      case SL_V: return cols(G.in.w, G.in.N, hk + kv * L.dim);
      case SL_G: return cols(G.in.w, G.in.N, hk + kv * (L.dim + (L.values_from_keys ? 0 : L.vdim)));
      case SL_Q_CONV: return upload_conv(m, G, 0, hk, host);
      case SL_K_CONV: return upload_conv(m, G, hk, kv * L.dim, host);
      case SL_Q_NORM: return norm(G.q_norm, false);
      case SL_K_NORM: return norm(G.k_norm, false);
      case SL_SINK: return vector(G.sink);
      case SL_REL: return upload_bias(m, L, G, host);
      default: break;
    }
  }
  if (L.mixer == MIX_GLA) {
    GlaDev& G = D.l;
    switch (t.slot) {
      case SL_Q: return cols(G.in.w, G.in.N, 0);
      case SL_K: return cols(G.in.w, G.in.N, hk);
      case SL_V: return cols(G.in.w, G.in.N, 2 * hk);
      case SL_V_GATE: return cols(G.in.w, G.in.N, 2 * hk + hv);
      case SL_A1: return cols(G.in.w, G.in.N, 2 * hk + 2 * hv);
      case SL_A2: return vector(G.a2);
      case SL_A2_B: return vector(G.a2_b);
      case SL_V_NORM: return norm(G.norm, false);
      default: break;
    }
  }
  switch (t.slot) {
    case SL_NORM1: return norm(D.ln1g, zc);
    case SL_NORM2: return norm(D.ln2g, zc);
    case SL_DQ_NORM: return norm(A.q_norm, false);
    case SL_DKV_NORM: return norm(A.kv_norm, false);
    case SL_DQ: return cols(A.in.w, A.in.N, 0);
    case SL_DKV: return cols(A.in.w, A.in.N, L.q_rank);
    case SL_G: return cols(A.in.w, A.in.N, (int64_t)L.q_rank + (L.kv_from < 0 ? L.kv_rank + L.rot_dim : 0));
    case SL_SINK: return vector(A.sink);
    case SL_UQ: return cols(A.uq.w, A.uq.N, 0);
    case SL_UK: return cols(A.ukv.w, A.ukv.N, 0);
    case SL_UV: return cols(A.ukv.w, A.ukv.N, (int64_t)L.heads * L.dim);
    case SL_O: return cols(D.o.w, m->dp, 0);
    case SL_GATE: return gate_up(D.gu.w, false, L.ffn);
    case SL_UP: return gate_up(D.gu.w, true, L.ffn);
    case SL_DOWN: return cols(D.down.w, m->dp, 0);
    case SL_ROUTER: return cols(D.x.router.w, D.x.router.N, 0);
    case SL_ROUTER_B: return vector(D.x.router.b);
    case SL_S_GATE: return gate_up(D.gu.w, false, L.shared_ffn);
    case SL_S_UP: return gate_up(D.gu.w, true, L.shared_ffn);
    case SL_S_DOWN: return cols(D.down.w, m->dp, 0);
    case SL_S_SG: return cols(D.x.router.w, D.x.router.N, L.experts);
    case SL_E_DOWN: return cols((char*)D.x.down + (size_t)t.expert * fp * m->dp * es, m->dp, 0);
    case SL_E_GATE: return gate_up((char*)D.x.gu + (size_t)t.expert * m->dp * 2 * fp * es, false, L.ffn);
    case SL_E_UP:
      if (D.x.gated) return gate_up((char*)D.x.gu + (size_t)t.expert * m->dp * 2 * fp * es, true, L.ffn);
      return cols((char*)D.x.gu + (size_t)t.expert * m->dp * fp * es, fp, 0);
    default: return fail("tensor slot not supported");
  }
}

int layered_init_random(rewb200_model* m, uint64_t seed, float std) {
  Ctx* c = m->c;
  const int dt = m->cfg.dtype;
  RB_REQUIRE(m->dp == m->cfg.d_model && m->vp == m->cfg.vocab, "random weights need a width and a vocabulary that are multiples of 8");
  uint64_t k = seed * 1000003ull;
  auto fill = [&](void* w, int64_t n) { return fill_normal_launch(c, w, dt, n, ++k, std); };
  RB_TRY(fill(m->embed, (int64_t)m->cfg.vocab * m->dp));
  RB_TRY(fill(m->lm.w, m->lm.K * m->lm.N));
  if (m->step_vec) RB_TRY(fill_normal_launch(c, m->step_vec, REWB200_F32, m->stack.loop_times * m->dp, ++k, std));
  RB_TRY(fill_const_launch(c, m->ng, REWB200_F32, m->dp, 1.f));
  for (LayerDev& D : m->layers) {
    RB_TRY(fill_const_launch(c, D.ln1g, REWB200_F32, m->dp, 1.f));
    if (D.ln2g) RB_TRY(fill_const_launch(c, D.ln2g, REWB200_F32, m->dp, 1.f));
    if (D.mixer == MIX_LATENT) {
      RB_TRY(fill_const_launch(c, D.a.q_norm, REWB200_F32, D.a.m.q_rank, 1.f));
      if (D.a.kv_norm) RB_TRY(fill_const_launch(c, D.a.kv_norm, REWB200_F32, D.a.m.kv_rank, 1.f));
    } else if (D.mixer == MIX_GQA) {
      if (D.g.q_norm) RB_TRY(fill_const_launch(c, D.g.q_norm, REWB200_F32, D.g.m.dim, 1.f));
      if (D.g.k_norm) RB_TRY(fill_const_launch(c, D.g.k_norm, REWB200_F32, D.g.m.dim, 1.f));
      if (D.g.conv) RB_TRY(fill_normal_launch(c, D.g.conv, REWB200_F32, D.g.m.taps * gqa_channels(D.g.m), ++k, 0.5f));
      if (D.g.bias) RB_TRY(fill_normal_launch(c, D.g.bias, REWB200_F32, (int64_t)D.g.m.heads * D.g.m.n_bias, ++k, 1.f));
    } else {
      RB_TRY(fill_const_launch(c, D.l.norm, REWB200_F32, D.l.m.vdim, 1.f));
      RB_TRY(fill_const_launch(c, D.l.a2_b, REWB200_F32, (int64_t)D.l.m.heads * D.l.m.dim, 2.f));
      RB_TRY(fill_normal_launch(c, D.l.a2, REWB200_F32, (int64_t)D.l.m.heads * D.l.m.dim * D.l.m.rank, ++k, std));
    }
    for (LinW* w : mixer_linears(D)) RB_TRY(fill(w->w, w->K * w->N));
    if (has_dense(D))
      for (LinW* w : {&D.gu, &D.down}) RB_TRY(fill(w->w, w->K * w->N));
    if (D.ff == 2) {
      RB_TRY(fill(D.x.router.w, D.x.router.K * D.x.router.N));
      RB_TRY(fill(D.x.gu, (int64_t)D.x.E * m->dp * (D.x.gated ? 2 : 1) * D.x.f));
      RB_TRY(fill(D.x.down, (int64_t)D.x.E * D.x.f * m->dp));
    }
  }
  RB_CUDA(cudaStreamSynchronize(c->stream));
  return REWB200_OK;
}

int layered_plans(rewb200_model* m) {
  if (m->cfg.dtype != REWB200_BF16) return REWB200_OK;
  auto plan = [&](LinW& w) { return linear_bf16_plan(&w.plan, (const bf16*)w.w, w.K, w.N, 0); };
  for (LayerDev& D : m->layers) {
    for (LinW* w : mixer_linears(D)) RB_TRY(plan(*w));
    if (has_dense(D))
      for (LinW* w : {&D.gu, &D.down}) RB_TRY(plan(*w));
    if (D.ff == 2) {
      RB_TRY(plan(D.x.router));
      RB_TRY(linear_bf16_plan(&D.x.plan_gu, (const bf16*)D.x.gu, m->dp, (D.x.gated ? 2 : 1) * D.x.f, D.x.E_l));
      RB_TRY(linear_bf16_plan(&D.x.plan_down, (const bf16*)D.x.down, D.x.f, m->dp, D.x.E_l));
    }
  }
  return plan(m->lm);
}

// Row-sized buffers of a layered step; called by ensure_acts after it has released the old ones.
int layered_acts(rewb200_session* s, int64_t rows) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  const size_t es = dtype_size(m->cfg.dtype);
  int64_t cq = 1, heads = 0;
  for (const LayerDev& D : m->layers) {
    cq = std::max(cq, D.a.uq.K);
    heads = std::max<int64_t>(heads, std::max(D.a.m.heads, D.g.m.heads));
  }
  heads = std::max<int64_t>(heads, 1);
  RB_TRY(acts_alloc(c, &s->xn2, (size_t)rows * m->dp * es));
  RB_TRY(acts_alloc(c, &s->cq, (size_t)rows * cq * es));
  RB_TRY(acts_alloc(c, (void**)&s->gate, (size_t)rows * heads * sizeof(float)));
  RB_TRY(acts_alloc(c, (void**)&s->part2, s->part_bytes));
  if (m->stack.block != BLOCK_OUTPUT_NORM && std::any_of(m->spec.begin(), m->spec.end(), [](const rewb200_layer& L) { return L.shared_ffn > 0; })) {
    RB_TRY(acts_alloc(c, (void**)&s->part3, s->part_bytes));
    RB_TRY(acts_alloc(c, (void**)&s->shared_gate, (size_t)rows * sizeof(float)));
  }
  if (c->record_layers) RB_TRY(acts_alloc(c, (void**)&s->layer_rec, m->runs.size() * (size_t)rows * m->dp * sizeof(float)));
  // padding columns are multiplied by zero weights, so they must hold finite values from the start
  RB_CUDA(cudaMemsetAsync(s->cq, 0, (size_t)rows * cq * es, c->stream));
  RB_CUDA(cudaMemsetAsync(s->attn, 0, (size_t)rows * m->nq * es, c->stream));
  RB_CUDA(cudaMemsetAsync(s->h, 0, (size_t)rows * std::max<int64_t>(std::max(m->max_ffn, m->max_moe_ffn), 1) * es, c->stream));
  return REWB200_OK;
}

// One cache of latents, of keys and values, or one recurrent state per lane, for every layer run that has its own.
int layered_session(rewb200_session* s, int64_t n_pages) {
  rewb200_model* m = s->m;
  const bool bf = m->cfg.dtype == REWB200_BF16;
  const size_t es = dtype_size(m->cfg.dtype);
  const size_t n = m->runs.size();
  s->kc.resize(n, nullptr);
  s->vc.resize(n, nullptr);
  s->tmK.resize(n);
  s->tmV.resize(n);
  s->state.resize(n, nullptr);
  auto zeroed = [&](void** p, size_t bytes) -> int {
    RB_CUDA(cudaMalloc(p, bytes));
    RB_CUDA(cudaMemsetAsync(*p, 0, bytes, m->c->stream));
    return REWB200_OK;
  };
  auto pages = [&](void** p, CUtensorMap* tm, int64_t rows, int64_t ld) -> int {
    RB_TRY(zeroed(p, (size_t)rows * ld * es));
    return bf ? make_tmap_2d_bf16(tm, *p, (uint64_t)ld, (uint64_t)rows, (uint64_t)ld * 2, 64, 64) : REWB200_OK;
  };
  for (size_t r = 0; r < n; ++r) {
    const LayerDev& D = m->layers[m->runs[r].layer];
    if (D.mixer == MIX_LATENT && D.a.m.own_kv) RB_TRY(pages(&s->kc[r], &s->tmK[r], n_pages * PAGE, D.a.ldc));
    if (D.mixer == MIX_GQA && D.g.m.own_kv) {
      RB_TRY(pages(&s->kc[r], &s->tmK[r], n_pages * D.g.m.kv_heads * PAGE, D.g.ldk));
      RB_TRY(pages(&s->vc[r], &s->tmV[r], n_pages * D.g.m.kv_heads * PAGE, D.g.ldv));
    }
    if (D.mixer == MIX_GQA && gqa_state_elems(D.g.m) > 0) RB_TRY(zeroed((void**)&s->state[r], (size_t)s->B * gqa_state_elems(D.g.m) * sizeof(float)));
    // a state needs no clearing between sequences: a portion that starts at position 0 does not read it
    if (D.mixer == MIX_GLA)
      RB_TRY(zeroed((void**)&s->state[r], (size_t)s->B * D.l.m.heads * D.l.m.dim * gla_state_ld(D.l.m.vdim) * sizeof(float)));
  }
  return REWB200_OK;
}

namespace {

// Rows of one lane an absorbed-attention tile covers at most.
constexpr int ABS_TILE_ROWS = 8;
// Rows of one lane a tile of the paged grouped-query kernel covers at most.
constexpr int GQA_TILE_ROWS = 16;
// Portions of at least this many tokens attend to keys and values expanded per head.  Expanding costs a Linear over the
// portion's keys, its own and its window's; the absorbed form costs (2 kv_rank + rot_dim) / (dim + rot_dim + vdim) times
// the score and value products of every query, on the slower mma.sync pipe.
constexpr int EXPAND_MIN_ROWS = 64;
// Portions of at least this many tokens run grouped-query attention on tcgen05 and gated linear attention in chunks.
constexpr int LARGE_MIN_ROWS = 64, CHUNK_MIN_ROWS = 32;

template <typename T>
int regrow(rewb200_session* s, T** p, size_t bytes) {
  Ctx* c = s->m->c;
  RB_CUDA(cudaStreamSynchronize(c->stream));
  if (s->graph) {
    cudaGraphExecDestroy(s->graph);
    s->graph = nullptr;
  }
  if (*p) {
    void* q = (void*)*p;
    *p = nullptr;
    RB_CUDA(cudaFree(q));
  }
  return acts_alloc(c, (void**)p, bytes);
}

}  // namespace

int layered_prepare(rewb200_session* s, const FwdOpts& o, int64_t rows) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  const size_t es = dtype_size(m->cfg.dtype);
  const bool uniform = o.entries == nullptr;
  RB_REQUIRE(!uniform || o.S == 1, "layered step: a step of several tokens per lane needs its portions");
  // ---- lists of the step: [row lane | row position | absorbed tiles | their chunks | expanded tiles | gathered keys |
  // chunks of gated linear attention | last rows of the portions | small and large tiles of grouped-query attention | small and
  // large portions of gated linear attention]
  int64_t abs_rows = rows, n_keys = 0;
  s->plan_host.clear();
  s->plan_abs_tiles = s->plan_chunks = s->plan_exp_tiles = s->plan_keys = s->plan_gla_chunks = s->plan_tails = 0;
  if (!uniform) {
    std::vector<int>& h = s->plan_host;
    h.assign(2 * rows, 0);
    std::vector<int2> tiles, chunks, keys;
    std::vector<ExpTile> exps;
    abs_rows = 0;
    int64_t reach = 0;  // the widest window of any layer, 0: everything
    const bool bf = m->cfg.dtype == REWB200_BF16;
    bool exp_ok = bf && c->latent_impl == 0, gqa_ok = bf && c->gqa_impl == 0, gla_ok = bf && c->gla_impl == 0;
    bool has_latent = false, has_gqa = false, has_gla = false;
    int taps = 0;           // of the longest convolution
    for (const LayerDev& D : m->layers) {
      if (D.mixer == MIX_GQA) {
        has_gqa = true;
        gqa_ok = gqa_ok && gqa_prefill_ok(D.g.m);
        taps = std::max(taps, D.g.m.taps);
      }
      if (D.mixer == MIX_GLA) {
        has_gla = true;
        gla_ok = gla_ok && gla_chunk_ok(D.l.m);
      }
      if (D.mixer != MIX_LATENT) continue;
      has_latent = true;
      exp_ok = exp_ok && latent_expanded_ok(D.a.m);
      reach = D.a.m.window == 0 ? INT32_MAX : std::max<int64_t>(reach, D.a.m.window);
    }
    std::vector<int2> gqa_small;
    std::vector<GqaTile> gqa_large;
    std::vector<GlaPortion> gla_small, gla_large;
    std::vector<int2> gla_chunk, tails;
    for (const StepEntry& e : *o.entries) {
      for (int i = 0; i < e.n; ++i) {
        h[e.row0 + i] = e.lane;
        h[rows + e.row0 + i] = e.pos0 + i;
      }
      for (int i = 0; i < std::min(taps - 1, e.n); ++i) tails.push_back(make_int2(e.row0 + e.n - 1 - i, i));
      if (has_gqa) {
        if (gqa_ok && e.n >= LARGE_MIN_ROWS)
          for (int i = 0; i < e.n; i += 256) gqa_large.push_back({e.row0 + i, std::min(256, e.n - i), e.pos0 + i, e.lane});
        else
          for (int i = 0; i < e.n; i += GQA_TILE_ROWS) gqa_small.push_back(make_int2(e.row0 + i, std::min(GQA_TILE_ROWS, e.n - i)));
      }
      if (has_gla) {
        const bool large = gla_ok && e.n >= CHUNK_MIN_ROWS;
        const GlaPortion p = {e.row0, e.n, e.pos0, e.lane, large ? (int)gla_chunk.size() : 0};
        (large ? gla_large : gla_small).push_back(p);
        if (large)
          for (int i = 0; i < gla_chunks(e.n); ++i) gla_chunk.push_back(gla_chunk_rows(p, i));
      }
      if (!has_latent) continue;
      if (exp_ok && e.n >= EXPAND_MIN_ROWS) {
        const int key0 = (int)std::max<int64_t>(0, (int64_t)e.pos0 - reach + 1);
        for (int i = 0; i < e.n; i += 256)
          exps.push_back({e.row0 + i, std::min(256, e.n - i), e.pos0 + i, key0, (int)keys.size() - key0, {0, 0, 0}});
        for (int p = key0; p < e.pos0 + e.n; ++p) keys.push_back(make_int2(e.lane, p));
        continue;
      }
      abs_rows = e.row0 + e.n;
      for (int i = 0; i < e.n; i += ABS_TILE_ROWS) tiles.push_back(make_int2(e.row0 + i, std::min(ABS_TILE_ROWS, e.n - i)));
      // the same rows in longer runs, whatever their lanes, for the per-head products around the attention
      for (int i = 0; i < e.n;) {
        const bool grow = !chunks.empty() && chunks.back().x + chunks.back().y == e.row0 + i && chunks.back().y < kChunkRows;
        const int room = grow ? kChunkRows - chunks.back().y : kChunkRows, k = std::min(room, e.n - i);
        if (grow) chunks.back().y += k;
        else chunks.push_back(make_int2(e.row0 + i, k));
        i += k;
      }
    }
    // long query tiles first: the last ones of a wave are then short
    std::stable_sort(exps.begin(), exps.end(), [](const ExpTile& x, const ExpTile& y) { return x.pos0 + x.n - x.key0 > y.pos0 + y.n - y.key0; });
    std::stable_sort(gqa_large.begin(), gqa_large.end(), [](const GqaTile& x, const GqaTile& y) { return x.pos0 + x.n > y.pos0 + y.n; });
    s->plan_gqa_small = (int)gqa_small.size();
    s->plan_gqa_large = (int)gqa_large.size();
    s->plan_gla_small = (int)gla_small.size();
    s->plan_gla_large = (int)gla_large.size();
    s->plan_gla_chunks = (int)gla_chunk.size();
    s->plan_tails = (int)tails.size();
    s->plan_abs_tiles = (int)tiles.size();
    s->plan_chunks = (int)chunks.size();
    s->plan_exp_tiles = (int)exps.size();
    s->plan_keys = (int)keys.size();
    n_keys = (int64_t)keys.size();
    auto append = [&](const void* p, size_t bytes) {
      const size_t at = h.size();
      h.resize(at + bytes / sizeof(int));
      if (bytes) memcpy(h.data() + at, p, bytes);
    };
    append(tiles.data(), tiles.size() * sizeof(int2));
    append(chunks.data(), chunks.size() * sizeof(int2));
    append(exps.data(), exps.size() * sizeof(ExpTile));
    append(keys.data(), keys.size() * sizeof(int2));
    append(gla_chunk.data(), gla_chunk.size() * sizeof(int2));
    append(tails.data(), tails.size() * sizeof(int2));
    append(gqa_small.data(), gqa_small.size() * sizeof(int2));
    append(gqa_large.data(), gqa_large.size() * sizeof(GqaTile));
    append(gla_small.data(), gla_small.size() * sizeof(GlaPortion));
    append(gla_large.data(), gla_large.size() * sizeof(GlaPortion));
    if (h.size() > s->plan_cap) {
      s->plan_cap = 0;
      RB_TRY(regrow(s, &s->plan_dev, h.size() * 2 * sizeof(int)));
      s->plan_cap = h.size() * 2;
    }
    RB_CUDA(cudaMemcpyAsync(s->plan_dev, h.data(), h.size() * sizeof(int), cudaMemcpyHostToDevice, c->stream));
  }
  if (n_keys > s->kvx_rows) {
    int64_t kv = 0, ldc = 0;
    for (const LayerDev& D : m->layers) {
      kv = std::max(kv, D.a.ukv.N);
      ldc = std::max(ldc, D.a.ldc);
    }
    s->kvx_rows = 0;
    RB_TRY(regrow(s, &s->kvx, (size_t)n_keys * kv * es));
    RB_TRY(regrow(s, &s->latx, (size_t)n_keys * ldc * es));
    // rows past a portion's last key are multiplied by zero probabilities: finite from the start
    RB_CUDA(cudaMemsetAsync(s->kvx, 0, (size_t)n_keys * kv * es, c->stream));
    RB_CUDA(cudaMemsetAsync(s->latx, 0, (size_t)n_keys * ldc * es, c->stream));
    s->kvx_rows = n_keys;
  }
  // ---- scratch of the absorbed path
  size_t chunk = 0;
  for (const LayerDev& D : m->layers)
    if (D.mixer == MIX_GLA) chunk = std::max(chunk, gla_chunk_bytes(D.l.m));
  if (chunk * s->plan_gla_chunks > s->gla_work_bytes) {
    s->gla_work_bytes = 0;
    RB_TRY(regrow(s, &s->gla_work, chunk * s->plan_gla_chunks));
    s->gla_work_bytes = chunk * s->plan_gla_chunks;
  }
  int64_t units = 0, stats = 0, qe = 0;
  int64_t g_units = 0, g_stats = 0;
  for (const LayerDev& D : m->layers) {
    if (D.mixer == MIX_GQA) {
      const int sp = gqa_kv_splits(c, D.g.m, uniform ? rows : s->plan_gqa_small, s->max_len);
      g_stats = std::max<int64_t>(g_stats, (int64_t)D.g.m.heads * sp);
      g_units = std::max<int64_t>(g_units, (int64_t)D.g.m.heads * sp * D.g.m.vdim);
    }
    if (D.mixer != MIX_LATENT) continue;
    const int64_t H = D.a.m.heads;
    const int sp = latent_kv_splits(c, D.a.m, rows, s->max_len);
    units = std::max(units, H * sp * D.a.m.kv_rank);
    stats = std::max(stats, H * sp);
    qe = std::max(qe, H * D.a.ldc);
  }
  if (rows * g_units > s->gqa_units) {
    s->gqa_units = 0;
    RB_TRY(regrow(s, &s->gqa_part, (size_t)rows * g_units * sizeof(float)));
    s->gqa_units = rows * g_units;
  }
  if (rows * g_stats > s->gqa_stats) {
    s->gqa_stats = 0;
    RB_TRY(regrow(s, &s->gqa_ml, (size_t)rows * g_stats * sizeof(float2)));
    s->gqa_stats = rows * g_stats;
  }
  if (abs_rows * units > s->abs_units) {
    s->abs_units = 0;
    RB_TRY(regrow(s, &s->olat, (size_t)abs_rows * units * sizeof(float)));
    s->abs_units = abs_rows * units;
  }
  if (abs_rows * stats > s->abs_stats) {
    s->abs_stats = 0;
    RB_TRY(regrow(s, &s->ml, (size_t)abs_rows * stats * sizeof(float2)));
    s->abs_stats = abs_rows * stats;
  }
  if (abs_rows * qe > s->abs_rows) {
    s->abs_rows = 0;
    RB_TRY(regrow(s, &s->qeff, (size_t)abs_rows * qe * es));
    RB_CUDA(cudaMemsetAsync(s->qeff, 0, (size_t)abs_rows * qe * es, c->stream));
    s->abs_rows = abs_rows * qe;
  }
  return REWB200_OK;
}

namespace {

// The lists of a step on the device (layered_prepare's upload, or none for a captured decode step).
struct StepLists {
  bool uniform = true;
  RowMap map = {};
  RowTiles abs = {}, chunks = {};
  const ExpTile* exp_tiles = nullptr;
  const int2 *key_list = nullptr, *gla_chunks = nullptr, *tails = nullptr;
  RowTiles gqa_small = {};
  const GqaTile* gqa_large = nullptr;
  const GlaPortion *gla_small = nullptr, *gla_large = nullptr;
};

StepLists step_lists(const rewb200_session* s, const FwdOpts& o, int64_t rows) {
  StepLists t;
  t.uniform = o.entries == nullptr;
  t.map = {nullptr, nullptr, s->d_pos, o.b0, o.S};
  t.abs = t.gqa_small = {nullptr, (int)rows, 1, 1};
  t.chunks = {nullptr, (int)((rows + kChunkRows - 1) / kChunkRows), 1, 1};
  if (t.uniform) return t;
  t.map.row_lane = s->plan_dev;
  t.map.row_pos = s->plan_dev + rows;
  t.abs.list = reinterpret_cast<const int2*>(s->plan_dev + 2 * rows);
  t.abs.count = s->plan_abs_tiles;
  t.chunks.list = t.abs.list + t.abs.count;
  t.chunks.count = s->plan_chunks;
  t.exp_tiles = reinterpret_cast<const ExpTile*>(t.chunks.list + t.chunks.count);
  t.key_list = reinterpret_cast<const int2*>(t.exp_tiles + s->plan_exp_tiles);
  t.gla_chunks = t.key_list + s->plan_keys;
  t.tails = t.gla_chunks + s->plan_gla_chunks;
  t.gqa_small.list = t.tails + s->plan_tails;
  t.gqa_small.count = s->plan_gqa_small;
  t.gqa_large = reinterpret_cast<const GqaTile*>(t.gqa_small.list + t.gqa_small.count);
  t.gla_small = reinterpret_cast<const GlaPortion*>(t.gqa_large + s->plan_gqa_large);
  t.gla_large = t.gla_small + s->plan_gla_small;
  return t;
}

// The mixers read s->xn and leave their output (ahead of the output projection) in s->attn.

int gqa_mixer(rewb200_session* s, const FwdOpts& o, const StepLists& t, size_t r, int64_t rows, bool in_graph) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  const int dt = m->cfg.dtype;
  const LayerRun& R = m->runs[r];
  LayerDev& D = m->layers[R.layer];
  GqaDev& G = D.g;
  const int64_t ldq = pad8((int64_t)G.m.heads * G.m.dim);
  int ks = 1;
  RB_TRY(run_linear(s, G.in, s->xn, m->dp, rows, true, 0, s->part, G.in.N, &ks));
  if (o.trace) RB_TRY(o.trace->mark(TC_QKV));
  GqaPostArgs pa;
  memset(&pa, 0, sizeof(pa));
  pa.m = G.m;
  pa.partial = s->part;
  pa.nsplit = ks;
  pa.split_stride = rows * G.in.N;
  pa.ld = G.in.N;
  pa.eps = m->cfg.eps;
  pa.map = t.map;
  pa.q = s->q;
  pa.ldq = ldq;
  pa.gate = s->gate;
  pa.kc = s->kc[R.cache];
  pa.vc = s->vc[R.cache];
  pa.ldk = G.ldk;
  pa.ldv = G.ldv;
  pa.block_table = s->block_table;
  pa.max_pages = s->max_pages;
  pa.capacity = s->max_len;
  pa.dtype = dt;
  pa.early = in_graph ? 1 : 0;
  pa.status = c->d_status;
  pa.state = s->state[r];
  pa.tails = t.tails;
  pa.n_tails = s->plan_tails;
  RB_TRY(gqa_post_launch(c, pa, rows));
  if (!t.uniform) RB_TRY(gqa_conv_state_launch(c, pa));
  if (o.trace) RB_TRY(o.trace->mark(TC_QKV_POST));
  GqaAttnArgs aa;
  memset(&aa, 0, sizeof(aa));
  aa.m = G.m;
  aa.map = t.map;
  aa.tiles = t.gqa_small;
  aa.max_tile_rows = t.uniform ? 1 : GQA_TILE_ROWS;
  aa.q = s->q;
  aa.ldq = ldq;
  aa.gate = s->gate;
  aa.out = s->attn;
  aa.ldo = D.o.K;
  aa.kc = pa.kc;
  aa.vc = pa.vc;
  if (dt == REWB200_BF16) {
    aa.tm_k = &s->tmK[R.cache];
    aa.tm_v = &s->tmV[R.cache];
  }
  aa.ldk = G.ldk;
  aa.ldv = G.ldv;
  aa.block_table = s->block_table;
  aa.max_pages = s->max_pages;
  aa.dtype = dt;
  aa.o_part = s->gqa_part;
  aa.ml = s->gqa_ml;
  aa.kv_splits = gqa_kv_splits(c, G.m, aa.tiles.count, s->max_len);
  aa.early_kv = in_graph ? 1 : 0;
  aa.status = c->d_status;
  RB_TRY(gqa_attn_launch(c, aa));
  if (!t.uniform && s->plan_gqa_large > 0) {
    GqaPrefillArgs fa;
    memset(&fa, 0, sizeof(fa));
    fa.m = G.m;
    fa.tiles = t.gqa_large;
    fa.count = s->plan_gqa_large;
    fa.q = (const bf16*)s->q;
    fa.ldq = ldq;
    fa.gate = s->gate;
    fa.out = (bf16*)s->attn;
    fa.ldo = D.o.K;
    fa.tm_k = aa.tm_k;
    fa.tm_v = aa.tm_v;
    fa.block_table = s->block_table;
    fa.max_pages = s->max_pages;
    fa.status = c->d_status;
    RB_TRY(gqa_prefill_launch(c, fa));
  }
  if (o.trace) RB_TRY(o.trace->mark(TC_ATTN));
  return REWB200_OK;
}

int gla_mixer(rewb200_session* s, const FwdOpts& o, const StepLists& t, size_t r, int64_t rows, bool in_graph) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  LayerDev& D = m->layers[m->runs[r].layer];
  GlaDev& A = D.l;
  int ks = 1;
  RB_TRY(run_linear(s, A.in, s->xn, m->dp, rows, true, 0, s->part, A.in.N, &ks));
  if (o.trace) RB_TRY(o.trace->mark(TC_QKV));
  GlaArgs ga;
  memset(&ga, 0, sizeof(ga));
  ga.m = A.m;
  ga.list = t.gla_small;
  ga.count = t.uniform ? (int)rows : s->plan_gla_small;
  ga.pos0 = s->d_pos;
  ga.b0 = o.b0;
  ga.partial = s->part;
  ga.nsplit = ks;
  ga.split_stride = rows * A.in.N;
  ga.ld = A.in.N;
  ga.eps = m->cfg.eps;
  ga.state = s->state[r];
  ga.ldv = (int)gla_state_ld(A.m.vdim);
  ga.out = s->attn;
  ga.ldo = D.o.K;
  ga.dtype = m->cfg.dtype;
  ga.early = in_graph ? 1 : 0;
  ga.status = c->d_status;
  RB_TRY(gla_recurrent_launch(c, ga));
  if (!t.uniform && s->plan_gla_large > 0) {
    ga.list = t.gla_large;
    ga.count = s->plan_gla_large;
    ga.chunks = t.gla_chunks;
    ga.n_chunks = s->plan_gla_chunks;
    ga.work = s->gla_work;
    RB_TRY(gla_chunk_launch(c, ga));
  }
  if (o.trace) RB_TRY(o.trace->mark(TC_ATTN));
  return REWB200_OK;
}

int latent_mixer(rewb200_session* s, const FwdOpts& o, const StepLists& t, size_t r, int64_t rows, bool in_graph) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  const int dt = m->cfg.dtype;
  const LayerRun& R = m->runs[r];
  LayerDev& D = m->layers[R.layer];
  LatentDev& A = D.a;
  const bool expand = !t.uniform && s->plan_exp_tiles > 0;
  int ks = 1;
  RB_TRY(run_linear(s, A.in, s->xn, m->dp, rows, true, 0, s->part, A.in.N, &ks));
  if (o.trace) RB_TRY(o.trace->mark(TC_QKV));
  LatentPostArgs pa;
  memset(&pa, 0, sizeof(pa));
  pa.m = A.m;
  pa.partial = s->part;
  pa.nsplit = ks;
  pa.split_stride = rows * A.in.N;
  pa.ld = A.in.N;
  pa.q_norm = A.q_norm;
  pa.kv_norm = A.kv_norm;
  pa.eps = m->cfg.eps;
  pa.map = t.map;
  pa.cq = s->cq;
  pa.ldcq = A.uq.K;
  pa.gate = s->gate;
  pa.cache = s->kc[R.cache];
  pa.block_table = s->block_table;
  pa.max_pages = s->max_pages;
  pa.capacity = s->max_len;
  pa.ldc = A.ldc;
  pa.dtype = dt;
  pa.early = in_graph ? 1 : 0;
  pa.status = c->d_status;
  RB_TRY(latent_post_launch(c, pa, rows));
  LatentAttnArgs aa;
  memset(&aa, 0, sizeof(aa));
  aa.m = A.m;
  aa.map = t.map;
  aa.tiles = t.abs;
  aa.chunks = t.chunks;
  aa.max_tile_rows = t.uniform ? 1 : ABS_TILE_ROWS;
  aa.rows = rows;
  if (expand) {
    RB_TRY(run_linear(s, A.uq, s->cq, A.uq.K, rows, false, EPI_BIAS_BF16, s->q, A.uq.N, nullptr));
    aa.q = s->q;
    aa.nsplit = 0;
  } else {
    RB_TRY(run_linear(s, A.uq, s->cq, A.uq.K, rows, true, 0, s->part, A.uq.N, &ks));
    aa.q = s->part;
    aa.nsplit = ks;
  }
  aa.split_stride = rows * A.uq.N;
  aa.ldq = A.uq.N;
  aa.ukv = A.ukv.w;
  aa.ld_ukv = A.ukv.N;
  aa.qeff = s->qeff;
  aa.olat = s->olat;
  aa.ml = s->ml;
  aa.kv_splits = latent_kv_splits(c, A.m, rows, s->max_len);
  aa.gate = s->gate;
  aa.out = s->attn;
  aa.ldo = D.o.K;
  aa.cache = s->kc[R.cache];
  aa.tm_cache = dt == REWB200_BF16 ? &s->tmK[R.cache] : nullptr;
  aa.block_table = s->block_table;
  aa.max_pages = s->max_pages;
  aa.ldc = A.ldc;
  aa.dtype = dt;
  aa.early_kv = in_graph ? 1 : 0;
  aa.status = c->d_status;
  if (o.trace) RB_TRY(o.trace->mark(TC_QKV_POST));
  RB_TRY(latent_attn_absorbed_launch(c, aa));
  if (expand) {
    LatentExpArgs ea;
    memset(&ea, 0, sizeof(ea));
    ea.m = A.m;
    ea.tiles = t.exp_tiles;
    ea.count = s->plan_exp_tiles;
    ea.q = (const bf16*)s->q;
    ea.ldq = A.uq.N;
    ea.gate = s->gate;
    ea.out = (bf16*)s->attn;
    ea.ldo = D.o.K;
    ea.kv = (const bf16*)s->kvx;
    ea.ldkv = A.ukv.N;
    ea.lat = (const bf16*)s->latx;
    ea.ldc = A.ldc;
    ea.keys = s->plan_keys;
    ea.status = c->d_status;
    RB_TRY(latent_gather_launch(c, (const bf16*)s->kc[R.cache], s->block_table, s->max_pages, A.ldc, t.key_list, (bf16*)s->latx, s->plan_keys));
    RB_TRY(linear_bf16_launch(c, A.ukv.plan, (const bf16*)s->latx, A.ldc, s->plan_keys, EPI_BIAS_BF16, 1, s->kvx, A.ukv.N, nullptr, nullptr, 0));
    RB_TRY(latent_attn_expanded_launch(c, ea));
  }
  if (o.trace) RB_TRY(o.trace->mark(TC_ATTN));
  return REWB200_OK;
}

int mixer(rewb200_session* s, const FwdOpts& o, const StepLists& t, size_t r, int64_t rows, bool in_graph) {
  switch (s->m->layers[s->m->runs[r].layer].mixer) {
    case MIX_GQA: return gqa_mixer(s, o, t, r, rows, in_graph);
    case MIX_GLA: return gla_mixer(s, o, t, r, rows, in_graph);
    default: return latent_mixer(s, o, t, r, rows, in_graph);
  }
}

// A gated SiLU feed-forward (dense, or the shared expert beside routed ones): f32 slabs of the result in `out`.
int dense_ff(rewb200_session* s, const FwdOpts& o, LayerDev& D, const void* x, int64_t rows, float* out, int* ks) {
  rewb200_model* m = s->m;
  const int64_t dp = m->dp;
  if (m->cfg.dtype == REWB200_BF16) {
    RB_TRY(run_linear(s, D.gu, x, dp, rows, false, EPI_SWIGLU_BF16, s->h, D.ffn_local, nullptr));
  } else {
    RB_TRY(run_linear(s, D.gu, x, dp, rows, false, EPI_BIAS_F32, s->gu32, 2 * D.ffn_local, nullptr));
    RB_TRY(swiglu_rows_f32_launch(m->c, s->gu32, (float*)s->h, rows, D.ffn_local));
  }
  if (o.trace) RB_TRY(o.trace->mark(TC_GATE_UP));
  RB_TRY(run_linear(s, D.down, s->h, D.ffn_local, rows, true, 0, out, dp, ks));
  if (o.trace) RB_TRY(o.trace->mark(TC_DOWN));
  return REWB200_OK;
}

// Runs `body` on the slot's second stream, after everything enqueued so far; the caller waits for c->ev_join.
template <typename F>
int on_side_stream(Ctx* c, F&& body) {
  RB_CUDA(cudaEventRecord(c->ev_fork, c->stream));
  RB_CUDA(cudaStreamWaitEvent(c->side, c->ev_fork, 0));
  cudaStream_t main_stream = c->stream;
  c->stream = c->side;
  const int st = body();
  c->stream = main_stream;
  RB_TRY(st);
  RB_CUDA(cudaEventRecord(c->ev_join, c->side));
  return REWB200_OK;
}

// Blocks normed on the way back: x += norm1(mixer(x)), x += norm2(ff(x)).
int output_norm_blocks(rewb200_session* s, const FwdOpts& o, const NormArgs& na, int64_t rows, bool in_graph) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  const int dt = m->cfg.dtype;
  const int64_t dp = m->dp;
  const StepLists t = step_lists(s, o, rows);
  OutputNormArgs base;
  memset(&base, 0, sizeof(base));
  base.x_res = s->x_res;
  base.split_stride = rows * dp;
  base.eps = m->cfg.eps;
  base.d = dp;
  base.d_mean = na.d_mean;
  base.out = s->xn;
  base.dtype = dt;
  base.status = c->d_status;
  if (o.trace) RB_TRY(o.trace->begin(c->stream));
  {
    OutputNormArgs a = base;
    a.embed = na.embed;
    a.ids = na.ids;
    a.vocab = na.vocab;
    RB_TRY(output_norm_launch(c, a, rows));
    if (o.trace) RB_TRY(o.trace->mark(TC_EMBED));
  }
  int moe_seen = 0;
  for (size_t r = 0; r < m->runs.size(); ++r) {
    LayerDev& D = m->layers[m->runs[r].layer];
    const bool last = r + 1 == m->runs.size();
    int ks_o = 1;
    RB_TRY(mixer(s, o, t, r, rows, in_graph));
    RB_TRY(run_linear(s, D.o, s->attn, D.o.K, rows, true, 0, s->part, dp, &ks_o));
    if (o.trace) RB_TRY(o.trace->mark(TC_O));
    {
      OutputNormArgs a = base;
      a.partial = s->part;
      a.nsplit = ks_o;
      a.gamma = D.ln1g;
      if (last && !D.ff) a.final_gamma = m->ng;
      RB_TRY(output_norm_launch(c, a, rows));
      if (o.trace) RB_TRY(o.trace->mark(TC_NORM_ATTN));
    }
    if (D.ff) {
      // slabs of a dense feed-forward or shared expert in part, the sum of the routed experts in part2
      OutputNormArgs a = base;
      const bool fork = D.ff == 2 && has_dense(D) && dt == REWB200_BF16 && rows <= 64 && c->moe_overlap && !o.trace;
      const bool pdl = c->use_pdl;
      auto dense = [&]() -> int { return dense_ff(s, o, D, s->xn, rows, s->part, &a.nsplit); };
      if (has_dense(D)) {
        a.partial = s->part;
        if (fork) {
          RB_TRY(on_side_stream(c, [&]() -> int {
            c->use_pdl = false;   // follows an event wait: plain launches
            const int st = dense();
            c->use_pdl = pdl;
            return st;
          }));
        } else {
          RB_TRY(dense());
        }
      }
      if (D.ff == 2) {
        RB_TRY(moe_routed(s, D.x, s->xn, dp, rows, false, s->part2, moe_seen++, false));
        a.partial2 = s->part2;
        a.nsplit2 = 1;
        if (o.trace) RB_TRY(o.trace->mark(TC_MOE));
      }
      if (fork) {
        RB_CUDA(cudaStreamWaitEvent(c->stream, c->ev_join, 0));
        c->use_pdl = false;       // two predecessors: a plain dependency
      }
      a.gamma = D.ln2g;
      if (last) a.final_gamma = m->ng;
      const int st = output_norm_launch(c, a, rows);
      c->use_pdl = pdl;
      RB_TRY(st);
      if (o.trace) RB_TRY(o.trace->mark(TC_NORM_FFN));
    }
    if (s->layer_rec && !t.uniform) {
      RB_CUDA(cudaMemcpyAsync(s->layer_rec + r * s->rows_cap * dp, s->x_res, (size_t)rows * dp * sizeof(float), cudaMemcpyDeviceToDevice, c->stream));
      s->layer_rows = rows;
    }
  }
  return REWB200_OK;
}

}  // namespace

// The layer runs of a layered model over `rows` rows; na carries the residual, the embedding and the ids.  Leaves the
// final norm's output in s->xn.
int layered_blocks(rewb200_session* s, const FwdOpts& o, const NormArgs& na, int64_t rows, bool in_graph) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  const int dt = m->cfg.dtype;
  const int64_t dp = m->dp;
  if (m->stack.block == BLOCK_OUTPUT_NORM) return output_norm_blocks(s, o, na, rows, in_graph);
  void* const ff_in = m->stack.block == BLOCK_ONE_NORM ? s->xn : s->xn2;   // what the feed-forward reads
  const StepLists t = step_lists(s, o, rows);
  auto ahead_of = [&](size_t r, NormArgs& a) {  // what the norm launch in front of run r adds and writes
    if (r == m->runs.size()) {
      a.gamma = m->ng;
      return;
    }
    const LayerRun& R = m->runs[r];
    const LayerDev& D = m->layers[R.layer];
    a.gamma = D.ln1g;
    if (D.ln2g) {
      a.gamma2 = D.ln2g;
      a.out2 = s->xn2;
    }
    if (R.step >= 0) a.add_vec = m->step_vec + (int64_t)R.step * dp;
    if (R.add_embed) {
      a.add_embed = 1;
    }
  };
  if (o.trace) RB_TRY(o.trace->begin(c->stream));
  {
    NormArgs a = na;
    ahead_of(0, a);
    a.add_embed = 0;
    RB_TRY(residual_norm_launch(c, a, rows));
    if (o.trace) RB_TRY(o.trace->mark(TC_EMBED));
  }
  int moe_seen = 0;
  for (size_t r = 0; r < m->runs.size(); ++r) {
    LayerDev& D = m->layers[m->runs[r].layer];
    int ks_o = 1, ks_f = 0, ks_s = 0;
    const bool fork = D.ff != 0 && dt == REWB200_BF16 && rows <= 64 && c->moe_overlap && !o.trace;
    const bool pdl = c->use_pdl;
    // ---- feed-forward branch: slabs in part2, those of a shared expert in part3
    auto ff_branch = [&]() -> int {
      if (D.ff == 0) return REWB200_OK;
      float* const keep = s->part;
      // beside the mixer both Linears are plain launches: a down projection launched early holds shared memory that the
      // mixer's short kernels then wait for (measured, 8B shape: 3.69 instead of 3.53 ms per step at batch 32)
      auto dense = [&](float* out, int* ks) -> int {
        s->part = out;   // scratch and slabs of this branch
        if (fork) c->use_pdl = false;
        const int st = dense_ff(s, o, D, ff_in, rows, out, ks);
        c->use_pdl = pdl;
        return st;
      };
      auto body = [&]() -> int {
        if (D.ff != 2) return dense(s->part2, &ks_f);
        s->part = s->part2;
        RB_TRY(moe_routed(s, D.x, ff_in, dp, rows, false, s->part2, moe_seen++, fork));
        ks_f = 1;
        if (o.trace) RB_TRY(o.trace->mark(TC_MOE));
        return has_dense(D) ? dense(s->part3, &ks_s) : REWB200_OK;
      };
      const int st = body();
      s->part = keep;
      return st;
    };
    if (fork) RB_TRY(on_side_stream(c, ff_branch));
    // ---- mixer
    RB_TRY(mixer(s, o, t, r, rows, in_graph));
    RB_TRY(run_linear(s, D.o, s->attn, D.o.K, rows, true, 0, s->part, dp, &ks_o));
    if (o.trace) RB_TRY(o.trace->mark(TC_O));
    if (!fork) RB_TRY(ff_branch());
    if (fork) RB_CUDA(cudaStreamWaitEvent(c->stream, c->ev_join, 0));
    // ---- both branches into the residual, norms of the next run
    NormArgs a = na;
    a.embed = nullptr;
    a.partial = s->part;
    a.nsplit = ks_o;
    a.split_stride = rows * dp;
    if (ks_f > 0) {
      a.partial2 = s->part2;
      a.nsplit2 = ks_f;
    }
    if (ks_s > 0) {
      a.partial3 = s->part3;
      a.nsplit3 = ks_s;
      a.scale3 = D.x.shared_gate ? s->shared_gate : nullptr;
    }
    ahead_of(r + 1, a);
    if (a.add_embed) a.embed = m->embed;
    if (fork) c->use_pdl = false;  // two predecessors: a plain dependency
    if (s->layer_rec && !t.uniform) {
      // the residual as the layer leaves it, ahead of what a loop adds
      NormArgs b = a;
      b.norm_kind = -1;
      b.add_embed = 0;
      b.embed = nullptr;
      b.add_vec = nullptr;
      b.gamma2 = nullptr;
      RB_TRY(residual_norm_launch(c, b, rows));
      RB_CUDA(cudaMemcpyAsync(s->layer_rec + r * s->rows_cap * dp, s->x_res, (size_t)rows * dp * sizeof(float), cudaMemcpyDeviceToDevice, c->stream));
      s->layer_rows = rows;
      a.partial = a.partial2 = a.partial3 = nullptr;
      a.nsplit = a.nsplit2 = a.nsplit3 = 0;
    }
    const int st = residual_norm_launch(c, a, rows);
    c->use_pdl = pdl;
    RB_TRY(st);
    if (o.trace) RB_TRY(o.trace->mark(TC_NORM_FFN));
  }
  return REWB200_OK;
}

}  // namespace rewb
