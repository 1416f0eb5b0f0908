// Layered models (rewb200_model_create_layers): weights, caches and the forward of decoders whose layers are described
// one by one.  They share the engine's sessions, lanes, page pool, captured decode step, sampler and lm_head
// (engine.cu); this file has what differs per layer.
//
// A block is the parallel x += mixer(norm1(x)) + ff(norm2(x)), where one launch (residual_norm) adds both branches' f32
// slabs to the residual, adds what a loop adds ahead of a pass, and leaves both norms of the next layer run, and in small
// steps the feed-forward branch runs on the slot's second stream beside the mixer; or x += norm1(mixer(x)), then
// x += norm2(ff(x)), where one launch (output_norm) per sublayer sums its slabs, norms the sum and adds it; or the parallel
// block with one norm that both branches read; or x += norm1b(mixer(norm1(x))), x += norm2b(ff(norm2(x))), where the same
// output_norm launch also leaves the next sublayer's norm, and a pass of a loop may open with a Linear over the stream and
// the embeddings side by side.
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
  SL_A2_B, SL_V_GATE, SL_V_NORM, SL_ROUTER_B, SL_S_GATE, SL_S_UP, SL_S_DOWN, SL_Q_CONV, SL_K_CONV, SL_S_SG,
  SL_BIGRAM, SL_LOOP_IN, SL_BACK1, SL_BACK2, SL_UP_B, SL_DOWN_B, SL_TALK, SL_Q_B, SL_K_B, SL_V_B, SL_V_CONV, SL_BETA, SL_ALPHA, SL_RATE, SL_DT_BIAS,
  SL_Y, SL_Y_B, SL_X, SL_X_B, SL_CONV, SL_CONV_B, SL_RA, SL_RI, SL_RA_B, SL_RI_B, SL_LAM
};
enum Block : int { BLOCK_PARALLEL = 0, BLOCK_OUTPUT_NORM = 1, BLOCK_ONE_NORM = 2, BLOCK_SANDWICH = 3 };
enum Sink : int { SINK_NONE = 0, SINK_LEARNED = 1, SINK_ONE = 2 };
enum Mixer : int { MIX_LATENT = 1, MIX_GQA = 2, MIX_GLA = 3, MIX_DELTA = 4, MIX_LRU = 5 };
struct TensorAt {
  Slot slot;
  int layer, expert;
  bool second = false;   // of the layer's second mixer
};
// The description of a layer's first or second mixer.
const rewb200_layer& mixer_spec(const rewb200_model* m, int layer, bool second) {
  return second ? m->spec[m->cfg.n_layers + m->spec[layer].beside - 1] : m->spec[layer];
}
bool has_loop_in(const rewb200_model* m) { return m->stack.loop_times > 0 && m->stack.loop_in; }

// The canonical tensors of a layered model (rew_b200/layered.py lists the same).
void tensors_of(const rewb200_model* m, std::vector<TensorAt>* out) {
  out->push_back({SL_EMBED, -1, -1});
  if (m->stack.bigram_buckets > 0) out->push_back({SL_BIGRAM, -1, -1});
  if (m->stack.loop_times > 0) out->push_back({has_loop_in(m) ? SL_LOOP_IN : SL_STEP, -1, -1});
  const bool sandwich = m->stack.block == BLOCK_SANDWICH;
  for (int l = 0; l < m->cfg.n_layers; ++l) {
    const rewb200_layer& L = m->spec[l];
    auto add = [&](std::initializer_list<Slot> slots) {
      for (Slot s : slots) out->push_back({s, l, -1});
    };
    add({SL_NORM1});
    if (sandwich) add({SL_BACK1});
    for (int k = 0; k < (L.beside ? 2 : 1); ++k) {
      const rewb200_layer& M = mixer_spec(m, l, k == 1);
      auto add = [&](std::initializer_list<Slot> slots) {
        for (Slot s : slots) out->push_back({s, l, -1, k == 1});
      };
      const bool own = M.kv_from < 0;
      if (M.mixer == MIX_LATENT) {
        add({SL_DQ, SL_DQ_NORM, SL_UQ});
        if (own) add({SL_DKV, SL_DKV_NORM});
        add({SL_UK, SL_UV});
        if (M.sink == SINK_LEARNED) add({SL_SINK});
      }
      if (M.mixer == MIX_GQA) {
        add({SL_Q});
        if (own) add({SL_K});
        if (own && !M.values_from_keys) add({SL_V});
        if (M.conv_taps > 0) add({SL_Q_CONV});
        if (M.conv_taps > 0 && own) add({SL_K_CONV});
        if (M.qk_norm) add({SL_Q_NORM});
        if (M.qk_norm && own) add({SL_K_NORM});
        if (M.bias_rows > 0) add({SL_REL});
        if (M.sink == SINK_LEARNED) add({SL_SINK});
        if (M.head_mix) add({SL_TALK});
        if (M.qkv_bias) add({SL_Q_B});
        if (M.qkv_bias && own) add({SL_K_B});
        if (M.qkv_bias && own && !M.values_from_keys) add({SL_V_B});
      }
      if (M.mixer == MIX_GLA) add({SL_Q, SL_K, SL_V, SL_A1, SL_A2, SL_A2_B, SL_V_GATE, SL_V_NORM});
      if (M.mixer == MIX_DELTA)
        add({SL_Q, SL_K, SL_V, SL_Q_CONV, SL_K_CONV, SL_V_CONV, SL_BETA, SL_ALPHA, SL_RATE, SL_DT_BIAS, SL_V_GATE, SL_V_NORM});
      if (M.mixer == MIX_LRU) add({SL_Y, SL_Y_B, SL_X, SL_X_B, SL_CONV, SL_CONV_B, SL_RA, SL_RI, SL_RA_B, SL_RI_B, SL_LAM});
      if (M.out_gate) add({SL_G});
      add({SL_O});
    }
    if (L.ff && m->stack.block != BLOCK_ONE_NORM) out->push_back({SL_NORM2, l, -1});
    if (L.ff && sandwich) add({SL_BACK2});
    if (L.ff == 1 && L.ff_act == 1) {
      add({SL_UP});
      if (L.ff_bias) add({SL_UP_B});
      add({SL_DOWN});
      if (L.ff_bias) add({SL_DOWN_B});
    } else if (L.ff == 1)
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
  const rewb200_layer* L = t.layer >= 0 ? &mixer_spec(m, t.layer, t.second) : nullptr;
  const bool grouped = L && (L->mixer == MIX_GQA || L->mixer == MIX_DELTA);   // kv_heads of keys
  *vec = false;
  auto mat = [&](int64_t r, int64_t c) { *rows = r; *cols = c; };
  auto v = [&](int64_t n) { *rows = 1; *cols = n; *vec = true; };
  switch (t.slot) {
    case SL_EMBED: mat(m->cfg.vocab, d); break;
    case SL_STEP: mat(m->stack.loop_times, d); break;
    case SL_BIGRAM: mat(m->stack.bigram_buckets + 1, d); break;
    case SL_LOOP_IN: mat(2 * d, d); break;
    case SL_FINAL: case SL_NORM1: case SL_NORM2: case SL_BACK1: case SL_BACK2: v(d); break;
    case SL_DQ: mat(d, L->q_rank); break;
    case SL_DQ_NORM: v(L->q_rank); break;
    case SL_UQ: mat(L->q_rank, (int64_t)L->heads * (L->dim + L->rot_dim)); break;
    case SL_DKV: mat(d, L->kv_rank + L->rot_dim); break;
    case SL_DKV_NORM: v(L->kv_rank); break;
    case SL_UK: mat(L->kv_rank, (int64_t)L->heads * L->dim); break;
    case SL_UV: mat(L->kv_rank, (int64_t)L->heads * L->vdim); break;
    case SL_G: mat(d, L->out_gate == 2 ? (int64_t)L->heads * L->vdim : L->heads); break;
    case SL_O: mat((int64_t)L->heads * L->vdim, d); break;
    case SL_GATE: case SL_UP: case SL_E_GATE: case SL_E_UP: mat(d, L->ffn); break;
    case SL_DOWN: case SL_E_DOWN: mat(L->ffn, d); break;
    case SL_ROUTER: mat(d, L->experts); break;
    case SL_ROUTER_B: v(L->experts); break;
    case SL_S_GATE: case SL_S_UP: mat(d, L->shared_ffn); break;
    case SL_S_DOWN: mat(L->shared_ffn, d); break;
    case SL_HEAD: mat(d, m->cfg.vocab); break;
    case SL_Q: mat(d, (int64_t)(L->mixer == MIX_DELTA ? L->kv_heads : L->heads) * L->dim); break;
    case SL_K: mat(d, (int64_t)(grouped ? L->kv_heads : L->heads) * L->dim); break;
    case SL_V: mat(d, (int64_t)(L->mixer == MIX_GQA ? L->kv_heads : L->heads) * L->vdim); break;
    case SL_Q_NORM: case SL_K_NORM: v(L->dim); break;
    case SL_REL: mat(L->bias_rows, L->heads); break;
    case SL_SINK: v(L->heads); break;
    case SL_A1: mat(d, L->decay_rank); break;
    case SL_A2: mat(L->decay_rank, (int64_t)L->heads * L->dim); break;
    case SL_A2_B: v((int64_t)L->heads * L->dim); break;
    case SL_V_GATE: mat(d, (int64_t)L->heads * L->vdim); break;
    case SL_V_NORM: v(L->vdim); break;
    case SL_Q_CONV: mat((int64_t)(L->mixer == MIX_DELTA ? L->kv_heads : L->heads) * L->dim, L->conv_taps); break;
    case SL_V_CONV: mat((int64_t)L->heads * L->vdim, L->conv_taps); break;
    case SL_UP_B: v(L->ffn); break;
    case SL_DOWN_B: v(d); break;
    case SL_TALK: mat(L->heads, L->heads); break;
    case SL_Q_B: case SL_Y_B: case SL_X_B: case SL_CONV_B: case SL_RA_B: case SL_RI_B: case SL_LAM: v((int64_t)L->heads * L->dim); break;
    case SL_K_B: v((int64_t)L->kv_heads * L->dim); break;
    case SL_V_B: v((int64_t)L->kv_heads * L->vdim); break;
    case SL_BETA: case SL_ALPHA: mat(d, L->heads); break;
    case SL_RATE: case SL_DT_BIAS: v(L->heads); break;
    case SL_Y: case SL_X: mat(d, (int64_t)L->heads * L->dim); break;
    case SL_CONV: mat((int64_t)L->heads * L->dim, L->conv_taps); break;
    case SL_RA: case SL_RI: mat((int64_t)L->heads * L->dim, L->dim); break;
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

// Convolution weights [taps][all] from the stored [channels][taps] of the channels from c0 on.
int upload_conv(rewb200_model* m, float* w, int taps, int64_t all, int64_t c0, int64_t channels, const float* host) {
  std::vector<float> t((size_t)taps * channels);
  for (int64_t ch = 0; ch < channels; ++ch)
    for (int j = 0; j < taps; ++j) t[(size_t)j * channels + ch] = host[ch * taps + j];
  RB_CUDA(cudaMemcpy2DAsync(w + c0, all * sizeof(float), t.data(), channels * sizeof(float), channels * sizeof(float), taps, cudaMemcpyHostToDevice,
                            m->c->stream));
  RB_CUDA(cudaStreamSynchronize(m->c->stream));
  return REWB200_OK;
}

// The Linear weights of a layer's mixer that are no routed experts (all of them padded matrices of the model dtype).
// The input projection of a layer's mixers; a second mixer's columns follow the first one's.
LinW& in_of(LayerDev& D) {
  return D.mixer == MIX_LATENT ? D.a.in : D.mixer == MIX_GQA ? D.g.in : D.mixer == MIX_GLA ? D.l.in : D.mixer == MIX_DELTA ? D.d.in : D.r.in;
}
std::vector<LinW*> mixer_linears(LayerDev& D) {
  if (D.mixer == MIX_LATENT) return {&D.a.in, &D.a.uq, &D.a.ukv, &D.o};
  return {&in_of(D), &D.o};
}
bool has(const LayerDev& D, int mixer) { return D.mixer == mixer || D.beside == mixer; }
bool has_dense(const LayerDev& D) { return D.ffn_local > 0; }

}  // namespace

int layered_create(rewb200_model* m, const rewb200_layer* layers, const rewb200_stack* stack) {
  const int n = m->cfg.n_layers;
  const size_t es = dtype_size(m->cfg.dtype);
  m->layered = true;
  RB_REQUIRE(stack->n_beside >= 0 && stack->n_beside <= n, "layered model: at most one second mixer a layer");
  m->spec.assign(layers, layers + n + stack->n_beside);
  m->stack = *stack;
  const rewb200_stack& st = m->stack;
  RB_REQUIRE(st.loop_times >= 0 && (st.loop_times == 0 || (st.loop_start >= 0 && st.loop_start < st.loop_stop && st.loop_stop <= n)),
             "layered model: the loop must cover layers start .. stop - 1 of the stack");
  RB_REQUIRE(st.block >= BLOCK_PARALLEL && st.block <= BLOCK_SANDWICH, "layered model: unknown block");
  RB_REQUIRE(st.block == BLOCK_SANDWICH || ((st.embed_scale == 0.f || st.embed_scale == 1.f) && st.bigram_buckets == 0 && !st.loop_in),
             "layered model: scaled embeddings, bigram tables and a Linear ahead of a pass belong to blocks normed on both sides");
  RB_REQUIRE(st.block != BLOCK_SANDWICH || st.loop_times == 0 || st.loop_in, "layered model: a loop of blocks normed on both sides opens with a Linear");
  RB_REQUIRE(st.bigram_buckets >= 0, "layered model: the bigram table must not have a negative size");
  RB_REQUIRE(st.block != BLOCK_OUTPUT_NORM || st.loop_times == 0, "layered model: blocks normed on the way back run without a loop");
  RB_REQUIRE(st.logit_softcap >= 0.f, "layered model: the cap of the logits must not be negative");
  std::vector<char> taken(st.n_beside, 0);
  for (int l = 0; l < n; ++l)
    for (int k = 0; k < (m->spec[l].beside ? 2 : 1); ++k) {
      const std::string who = "layer " + std::to_string(l) + ": ";
      if (k == 1) {
        const int b = m->spec[l].beside;
        RB_REQUIRE(b > 0 && b <= st.n_beside && !taken[b - 1], who + "no such second mixer");
        taken[b - 1] = 1;
        const int first = m->spec[l].mixer, second = m->spec[n + b - 1].mixer;
        RB_REQUIRE((second == MIX_DELTA || second == MIX_LRU) && first != second && first != MIX_LATENT, who + "these mixers do not stand beside one another");
      }
      const rewb200_layer& L = mixer_spec(m, l, k == 1);
      RB_REQUIRE(L.mixer >= MIX_LATENT && L.mixer <= MIX_LRU, who + "unknown mixer");
      RB_REQUIRE(L.heads > 0 && L.dim > 0 && L.vdim > 0, who + "mixer sizes must be positive");
      RB_REQUIRE(L.sink >= SINK_NONE && L.sink <= SINK_ONE, who + "unknown sink");
      RB_REQUIRE(L.out_gate >= 0 && L.out_gate <= (L.mixer == MIX_GQA ? 2 : L.mixer == MIX_LATENT ? 1 : 0), who + "unknown output gate");
      RB_REQUIRE(L.mixer == MIX_GQA || (!L.values_from_keys && !L.qkv_bias && !L.rope_pairs && !L.v_norm && !L.keep_first && !L.head_mix),
                 who + "biases, values from keys, neighbouring pairs, normed values, kept keys and mixed heads belong to grouped-query attention");
      RB_REQUIRE(L.conv_taps >= 0 && (L.mixer == MIX_GQA || L.mixer >= MIX_DELTA || L.conv_taps == 0), who + "this mixer has no convolution");
      RB_REQUIRE(L.mix_scale == 0.f || L.mix_scale == 1.f || L.mixer == MIX_GQA || L.mixer >= MIX_DELTA, who + "this mixer's output has no factor");
      if (L.kv_from >= 0) {
        RB_REQUIRE((L.mixer == MIX_LATENT || L.mixer == MIX_GQA) && L.kv_from < l, who + "kv_from must name an earlier layer");
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
        RB_REQUIRE(!L.qkv_bias || (L.conv_taps == 0 && !L.values_from_keys), who + "biases and a convolution, or values that are keys, do not go together");
        RB_REQUIRE(L.window >= 0 && L.keep_first >= 0 && (L.window > 0 || L.keep_first == 0), who + "kept first keys need a window");
      } else if (L.mixer == MIX_GLA) {
        RB_REQUIRE(L.decay_rank > 0 && L.tau > 0.f, who + "decay_rank and tau must be positive");
      } else if (L.mixer == MIX_DELTA) {
        RB_REQUIRE(L.kv_heads > 0 && L.heads % L.kv_heads == 0 && L.conv_taps > 0, who + "the delta rule needs a convolution and heads divisible by kv_heads");
      } else {
        RB_REQUIRE(L.vdim == L.dim && L.conv_taps > 0 && L.heads <= 256, who + "a linear recurrent unit needs a convolution and at most 256 blocks");
      }
    }
  for (int l = 0; l < n; ++l) {
    const rewb200_layer& L = m->spec[l];
    const std::string who = "layer " + std::to_string(l) + ": ";
    RB_REQUIRE(L.ff_act >= 0 && L.ff_act <= 1 && (L.ff_act == 0 || L.ff == 1), who + "unknown activation");
    RB_REQUIRE(!L.ff_bias || (L.ff_act == 1 && st.block == BLOCK_SANDWICH), who + "biases of the feed-forward belong to one without a gate in blocks normed on both sides");
    RB_REQUIRE(st.block != BLOCK_SANDWICH || L.ff <= 1, who + "blocks normed on both sides have a dense feed-forward or none");
    RB_REQUIRE(L.ff >= 0 && L.ff <= 2 && (L.ff == 0 || L.ffn > 0), who + "unknown feed-forward");
    RB_REQUIRE(L.shared_ffn >= 0 && (L.ff == 2 || L.shared_ffn == 0), who + "a shared expert stands beside routed ones");
    RB_REQUIRE(!L.shared_gate || (L.shared_ffn > 0 && st.block != BLOCK_OUTPUT_NORM), who + "the gate of a shared expert needs one, in a parallel block");
    RB_REQUIRE(L.ff != 2 || (L.experts > 0 && L.experts <= 256 && L.top_k > 0 && L.top_k <= L.experts),
               who + "experts must be in 1..256 and top in 1..experts");
  }
  const int64_t d = m->cfg.d_model, dp = m->dp = pad8(d);
  m->vp = pad8(m->cfg.vocab);
  RB_TRY(zero_weights(m, &m->embed, (size_t)m->cfg.vocab * dp * es));
  if (st.bigram_buckets > 0) RB_TRY(zero_weights(m, &m->bigram, ((size_t)st.bigram_buckets + 1) * dp * es));
  if (has_loop_in(m)) RB_TRY(zero_lin(m, &m->loop_in, 2 * dp, dp));
  else if (st.loop_times > 0) RB_TRY(zero_weights(m, (void**)&m->step_vec, (size_t)st.loop_times * dp * sizeof(float)));
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
  auto f32 = [&](float** p, int64_t count) { return zero_weights(m, (void**)p, (size_t)count * sizeof(float)); };
  auto scale_of = [](const rewb200_layer& L) { return L.mix_scale == 0.f ? 1.f : L.mix_scale; };
  // The parts of a delta rule or recurrent unit but the input projection, whose columns it returns.
  auto delta_of = [&](const rewb200_layer& L, DeltaDev& A, int64_t* cols) -> int {
    const int64_t hv = (int64_t)L.heads * L.vdim;
    RB_TRY(f32(&A.rate, L.heads));
    RB_TRY(f32(&A.dt_bias, L.heads));
    RB_TRY(f32(&A.norm, L.vdim));
    A.m = DeltaDims{L.heads, L.kv_heads, L.dim, L.vdim, A.rate, A.dt_bias, A.norm, scale_of(L)};
    const int64_t ch = delta_channels(A.m);
    RB_TRY(f32(&A.w, L.conv_taps * ch));
    A.conv = ConvDims{ch, L.conv_taps, A.w, nullptr, nullptr, 1};
    *cols = ch + hv + 2 * L.heads;
    return REWB200_OK;
  };
  auto lru_of = [&](const rewb200_layer& L, LruDev& A, int64_t* cols) -> int {
    const int64_t w = (int64_t)L.heads * L.dim, ldn = pad8(L.dim);
    for (float** p : {&A.x_bias, &A.conv_bias, &A.y_bias, &A.decay}) RB_TRY(f32(p, w));
    RB_TRY(f32(&A.w, L.conv_taps * w));
    RB_TRY(f32(&A.gate_bias, L.heads * 2 * ldn));
    RB_TRY(zero_weights(m, &A.gates, (size_t)L.heads * ldn * 2 * ldn * es));
    A.m = LruDims{L.heads, L.dim, (int)ldn, A.decay, A.y_bias, scale_of(L)};
    A.conv = ConvDims{w, L.conv_taps, A.w, A.x_bias, A.conv_bias, 0};
    *cols = 2 * w;
    return REWB200_OK;
  };
  m->layers.resize(n);
  int64_t widest = dp, q_cols = 0, attn_cols = 0;
  for (int l = 0; l < n; ++l) {
    const rewb200_layer& L = m->spec[l];
    LayerDev& D = m->layers[l];
    D.mixer = L.mixer;
    RB_TRY(zero_weights(m, (void**)&D.ln1g, dp * sizeof(float)));
    if (L.ff && st.block != BLOCK_ONE_NORM) RB_TRY(zero_weights(m, (void**)&D.ln2g, dp * sizeof(float)));
    if (st.block == BLOCK_SANDWICH) RB_TRY(f32(&D.back1, dp));
    if (st.block == BLOCK_SANDWICH && L.ff) RB_TRY(f32(&D.back2, dp));
    const bool own = L.kv_from < 0;
    int64_t beside_cols = 0;   // of the second mixer in the input projection
    if (L.beside) {
      const rewb200_layer& M = mixer_spec(m, l, true);
      D.beside = M.mixer;
      RB_TRY(M.mixer == MIX_DELTA ? delta_of(M, D.d, &beside_cols) : lru_of(M, D.r, &beside_cols));
    }
    // the projection for `cols` columns of the first mixer and those of the second
    auto in_lin = [&](LinW* w, int64_t cols) -> int {
      D.beside_in = pad8(cols);
      RB_TRY(zero_lin(m, w, dp, D.beside_in + pad8(beside_cols)));
      widest = std::max(widest, w->N);
      return REWB200_OK;
    };
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
      G.gate_col = (int64_t)L.heads * L.dim + (own ? (int64_t)L.kv_heads * (L.dim + (L.values_from_keys ? 0 : L.vdim)) : 0);
      RB_TRY(in_lin(&G.in, G.gate_col + (L.out_gate == 2 ? (int64_t)L.heads * L.vdim : L.out_gate ? L.heads : 0)));
      if (L.qkv_bias) RB_TRY(f32(&G.in_bias, G.gate_col));
      if (L.head_mix) RB_TRY(f32(&G.talk, (int64_t)L.heads * L.heads));
      if (L.qk_norm) RB_TRY(zero_weights(m, (void**)&G.q_norm, L.dim * sizeof(float)));
      if (L.qk_norm && own) RB_TRY(zero_weights(m, (void**)&G.k_norm, L.dim * sizeof(float)));
      const int nb = L.bias_rows > 0 ? bias_distances(L.bias_rows, L.bias_max) : 0;
      if (nb > 0) RB_TRY(zero_weights(m, (void**)&G.bias, (size_t)L.heads * nb * sizeof(float)));
      RB_TRY(sink_of(L, &G.sink));
      G.m = GqaDims{L.heads, L.kv_heads, L.dim, L.vdim, own ? 1 : 0, L.out_gate == 1, L.scale, G.q_norm, G.k_norm, L.temp_every, L.temp_coef, G.bias, nb, G.sink,
                    L.values_from_keys, L.conv_taps, nullptr, L.rope_dims, nullptr, L.rope_pairs, L.v_norm, G.in_bias, L.window, L.keep_first, G.talk,
                    0, L.out_gate == 2, scale_of(L)};
      RB_TRY(rope_of(L, &G.m.rope));
      if (L.conv_taps > 0) RB_TRY(zero_weights(m, (void**)&G.conv, (size_t)L.conv_taps * gqa_channels(G.m) * sizeof(float)));
      G.m.conv = G.conv;
      q_cols = std::max(q_cols, pad8((int64_t)L.heads * L.dim));
    } else if (L.mixer == MIX_DELTA) {
      int64_t cols = 0;
      RB_TRY(delta_of(L, D.d, &cols));
      RB_TRY(in_lin(&D.d.in, cols));
    } else if (L.mixer == MIX_LRU) {
      int64_t cols = 0;
      RB_TRY(lru_of(L, D.r, &cols));
      RB_TRY(in_lin(&D.r.in, cols));
    } else {
      GlaDev& A = D.l;
      const int64_t hk = (int64_t)L.heads * L.dim, hv = (int64_t)L.heads * L.vdim;
      RB_TRY(in_lin(&A.in, 2 * hk + 2 * hv + L.decay_rank));
      RB_TRY(zero_weights(m, (void**)&A.a2, hk * L.decay_rank * sizeof(float)));
      RB_TRY(zero_weights(m, (void**)&A.a2_b, hk * sizeof(float)));
      RB_TRY(zero_weights(m, (void**)&A.norm, L.vdim * sizeof(float)));
      A.m = GlaDims{L.heads, L.dim, L.vdim, L.decay_rank, L.tau, A.a2, A.a2_b, A.norm};
    }
    D.beside_out = pad8((int64_t)L.heads * L.vdim);
    const rewb200_layer& M = mixer_spec(m, l, D.beside != 0);
    RB_TRY(zero_lin(m, &D.o, D.beside_out + (D.beside ? pad8((int64_t)M.heads * M.vdim) : 0), dp));
    attn_cols = std::max(attn_cols, D.o.K);
    D.ff = L.ff;
    const int64_t fp = pad8(L.ffn);
    if (L.ff == 1) {
      D.ffn_local = fp;
      D.gelu = L.ff_act == 1;
      m->max_ffn = std::max(m->max_ffn, fp);
      RB_TRY(zero_lin(m, &D.gu, dp, D.gelu ? fp : 2 * fp));
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
    if (L.kv_from >= 0)   // the latest run of that layer: in a loop, the one of the same pass
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
  if (t.slot == SL_BIGRAM) return cols(m->bigram, m->dp, 0);
  if (t.slot == SL_LOOP_IN) {   // the rows of x, then those of the embeddings
    const int64_t d = R / 2;
    RB_TRY(scatter(m, C, 0, 0, d, C, m->loop_in.w, true, m->dp, C, C, 0));
    return scatter(m, C, d, 0, d, C, (char*)m->loop_in.w + (size_t)m->dp * m->dp * es, true, m->dp, C, C, 0);
  }
  if (t.slot == SL_STEP) return scatter(m, C, 0, 0, R, C, m->step_vec, false, m->dp, C, C, 0);
  if (t.slot == SL_FINAL) return norm(m->ng, zc);
  if (t.slot == SL_HEAD) return cols(m->lm.w, m->vp, 0);
  LayerDev& D = m->layers[t.layer];
  const rewb200_layer& L = mixer_spec(m, t.layer, t.second);
  LatentDev& A = D.a;
  const int64_t in0 = t.second ? D.beside_in : 0;
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
      case SL_G: return cols(G.in.w, G.in.N, G.gate_col);
      case SL_Q_CONV: return upload_conv(m, G.conv, G.m.taps, gqa_channels(G.m), 0, hk, host);
      case SL_K_CONV: return upload_conv(m, G.conv, G.m.taps, gqa_channels(G.m), hk, kv * L.dim, host);
      case SL_TALK: return vector(G.talk);
      case SL_Q_B: return vector(G.in_bias);
      case SL_K_B: return vector(G.in_bias + hk);
      case SL_V_B: return vector(G.in_bias + hk + kv * L.dim);
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
  if (L.mixer == MIX_DELTA) {
    DeltaDev& G = D.d;
    LinW& in = in_of(D);
    const int64_t gk = (int64_t)L.kv_heads * L.dim, ch = G.conv.channels;
    auto conv = [&](int64_t c0, int64_t n) { return upload_conv(m, G.w, L.conv_taps, ch, c0, n, host); };
    switch (t.slot) {
      case SL_Q: return cols(in.w, in.N, in0);
      case SL_K: return cols(in.w, in.N, in0 + gk);
      case SL_V: return cols(in.w, in.N, in0 + 2 * gk);
      case SL_V_GATE: return cols(in.w, in.N, in0 + ch);
      case SL_BETA: return cols(in.w, in.N, in0 + ch + hv);
      case SL_ALPHA: return cols(in.w, in.N, in0 + ch + hv + L.heads);
      case SL_Q_CONV: return conv(0, gk);
      case SL_K_CONV: return conv(gk, gk);
      case SL_V_CONV: return conv(2 * gk, hv);
      case SL_RATE:
        RB_TRY(vector(G.rate));
        return delta_rate_launch(m->c, G.rate, L.heads);
      case SL_DT_BIAS: return vector(G.dt_bias);
      case SL_V_NORM: return norm(G.norm, false);
      default: break;
    }
  }
  if (L.mixer == MIX_LRU) {
    LruDev& G = D.r;
    LinW& in = in_of(D);
    const int64_t ldn = G.m.ldn;
    // a gate's matrices [out, in] per block, transposed into [in][r | i]
    auto gate = [&](int64_t off) -> int {
      const int64_t n = L.dim;
      std::vector<float> w((size_t)(L.heads * n * n));
      for (int64_t b = 0; b < L.heads; ++b)
        for (int64_t o = 0; o < n; ++o)
          for (int64_t i = 0; i < n; ++i) w[(b * n + i) * n + o] = host[(b * n + o) * n + i];
      RB_TRY(upload_stage(m, w.data(), numel));
      for (int64_t b = 0; b < L.heads; ++b)
        RB_TRY(scatter(m, n, b * n, 0, n, n, (char*)G.gates + (size_t)b * ldn * 2 * ldn * es, true, 2 * ldn, n, n, off));
      return REWB200_OK;
    };
    auto gate_bias = [&](int64_t off) { return scatter(m, L.dim, 0, 0, L.heads, L.dim, G.gate_bias + off, false, 2 * ldn, L.dim, L.dim, 0); };
    switch (t.slot) {
      case SL_Y: return cols(in.w, in.N, in0);
      case SL_X: return cols(in.w, in.N, in0 + hk);
      case SL_Y_B: return vector(G.y_bias);
      case SL_X_B: return vector(G.x_bias);
      case SL_CONV: return upload_conv(m, G.w, L.conv_taps, hk, 0, hk, host);
      case SL_CONV_B: return vector(G.conv_bias);
      case SL_RA: return gate(0);
      case SL_RI: return gate(ldn);
      case SL_RA_B: return gate_bias(0);
      case SL_RI_B: return gate_bias(ldn);
      case SL_LAM:
        RB_TRY(vector(G.decay));
        return lru_decay_launch(m->c, G.decay, hk);
      default: break;
    }
  }
  switch (t.slot) {
    case SL_NORM1: return norm(D.ln1g, zc);
    case SL_NORM2: return norm(D.ln2g, zc);
    case SL_BACK1: return norm(D.back1, zc);
    case SL_BACK2: return norm(D.back2, zc);
    case SL_UP_B: return vector(D.gu.b);
    case SL_DOWN_B: return vector(D.down.b);
    case SL_DQ_NORM: return norm(A.q_norm, false);
    case SL_DKV_NORM: return norm(A.kv_norm, false);
    case SL_DQ: return cols(A.in.w, A.in.N, 0);
    case SL_DKV: return cols(A.in.w, A.in.N, L.q_rank);
    case SL_G: return cols(A.in.w, A.in.N, (int64_t)L.q_rank + (L.kv_from < 0 ? L.kv_rank + L.rot_dim : 0));
    case SL_SINK: return vector(A.sink);
    case SL_UQ: return cols(A.uq.w, A.uq.N, 0);
    case SL_UK: return cols(A.ukv.w, A.ukv.N, 0);
    case SL_UV: return cols(A.ukv.w, A.ukv.N, (int64_t)L.heads * L.dim);
    case SL_O: return cols((char*)D.o.w + (size_t)(t.second ? D.beside_out : 0) * m->dp * es, m->dp, 0);
    case SL_GATE: return gate_up(D.gu.w, false, L.ffn);
    case SL_UP: return D.gelu ? cols(D.gu.w, D.gu.N, 0) : gate_up(D.gu.w, true, L.ffn);
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
  if (m->bigram) RB_TRY(fill(m->bigram, ((int64_t)m->stack.bigram_buckets + 1) * m->dp));
  if (m->loop_in.w) RB_TRY(fill(m->loop_in.w, m->loop_in.K * m->loop_in.N));
  if (m->step_vec) RB_TRY(fill_normal_launch(c, m->step_vec, REWB200_F32, m->stack.loop_times * m->dp, ++k, std));
  RB_TRY(fill_const_launch(c, m->ng, REWB200_F32, m->dp, 1.f));
  for (LayerDev& D : m->layers) {
    RB_TRY(fill_const_launch(c, D.ln1g, REWB200_F32, m->dp, 1.f));
    if (D.ln2g) RB_TRY(fill_const_launch(c, D.ln2g, REWB200_F32, m->dp, 1.f));
    for (float* p : {D.back1, D.back2})
      if (p) RB_TRY(fill_const_launch(c, p, REWB200_F32, m->dp, 1.f));
    if (has(D, MIX_DELTA)) {
      RB_TRY(fill_normal_launch(c, D.d.w, REWB200_F32, D.d.conv.taps * D.d.conv.channels, ++k, 0.5f));
      RB_TRY(fill_const_launch(c, D.d.rate, REWB200_F32, D.d.m.heads, 0.05f));
      RB_TRY(fill_const_launch(c, D.d.norm, REWB200_F32, D.d.m.vdim, 1.f));
    }
    if (has(D, MIX_LRU)) {
      const int64_t w = (int64_t)D.r.m.blocks * D.r.m.n;
      RB_REQUIRE(D.r.m.n == D.r.m.ldn, "random weights need blocks of a multiple of 8 channels");
      RB_TRY(fill_normal_launch(c, D.r.w, REWB200_F32, D.r.conv.taps * w, ++k, 0.5f));
      RB_TRY(fill_const_launch(c, D.r.decay, REWB200_F32, w, -0.1f));
      RB_TRY(fill(D.r.gates, (int64_t)D.r.m.blocks * D.r.m.n * 2 * D.r.m.n));
    }
    if (D.mixer == MIX_LATENT) {
      RB_TRY(fill_const_launch(c, D.a.q_norm, REWB200_F32, D.a.m.q_rank, 1.f));
      if (D.a.kv_norm) RB_TRY(fill_const_launch(c, D.a.kv_norm, REWB200_F32, D.a.m.kv_rank, 1.f));
    } else if (D.mixer == MIX_GQA) {
      if (D.g.q_norm) RB_TRY(fill_const_launch(c, D.g.q_norm, REWB200_F32, D.g.m.dim, 1.f));
      if (D.g.k_norm) RB_TRY(fill_const_launch(c, D.g.k_norm, REWB200_F32, D.g.m.dim, 1.f));
      if (D.g.conv) RB_TRY(fill_normal_launch(c, D.g.conv, REWB200_F32, D.g.m.taps * gqa_channels(D.g.m), ++k, 0.5f));
      if (D.g.bias) RB_TRY(fill_normal_launch(c, D.g.bias, REWB200_F32, (int64_t)D.g.m.heads * D.g.m.n_bias, ++k, 1.f));
      if (D.g.talk) RB_TRY(fill_normal_launch(c, D.g.talk, REWB200_F32, (int64_t)D.g.m.heads * D.g.m.heads, ++k, 0.3f));
    } else if (D.mixer == MIX_GLA) {
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
  for (LayerDev& D : m->layers)
    if (D.g.talk) {
      D.g.talk_host.resize((size_t)D.g.m.heads * D.g.m.heads);
      RB_CUDA(cudaMemcpyAsync(D.g.talk_host.data(), D.g.talk, D.g.talk_host.size() * sizeof(float), cudaMemcpyDeviceToHost, m->c->stream));
      RB_CUDA(cudaStreamSynchronize(m->c->stream));
      D.g.m.talk_wide = std::any_of(D.g.talk_host.begin(), D.g.talk_host.end(), [](float t) { return !(std::fabs(t) < 65504.f); });
    }
  if (m->cfg.dtype != REWB200_BF16) return REWB200_OK;
  auto plan = [&](LinW& w) { return linear_bf16_plan(&w.plan, (const bf16*)w.w, w.K, w.N, 0); };
  if (m->loop_in.w) RB_TRY(plan(m->loop_in));
  for (LayerDev& D : m->layers) {
    for (LinW* w : mixer_linears(D)) RB_TRY(plan(*w));
    if (has(D, MIX_LRU)) RB_TRY(linear_bf16_plan(&D.r.plan_gates, (const bf16*)D.r.gates, D.r.m.ldn, 2 * D.r.m.ldn, D.r.m.blocks));
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
  int64_t conv = 0, gates = 0, blocks = 0;
  for (const LayerDev& D : m->layers) {
    if (has(D, MIX_DELTA)) conv = std::max(conv, pad8(D.d.conv.channels));
    if (!has(D, MIX_LRU)) continue;
    conv = std::max<int64_t>(conv, (int64_t)D.r.m.blocks * D.r.m.ldn);
    gates = std::max<int64_t>(gates, (int64_t)D.r.m.blocks * 2 * D.r.m.ldn);
    blocks = std::max<int64_t>(blocks, D.r.m.blocks);
  }
  auto zeroed = [&](void** p, size_t bytes) -> int {
    RB_TRY(acts_alloc(c, p, bytes));
    RB_CUDA(cudaMemsetAsync(*p, 0, bytes, c->stream));
    return REWB200_OK;
  };
  if (conv) RB_TRY(zeroed(&s->conv, (size_t)rows * conv * es));
  if (gates) RB_TRY(zeroed((void**)&s->gate_pre, (size_t)rows * gates * sizeof(float)));
  if (gates) RB_TRY(zeroed((void**)&s->group_rows, (size_t)(blocks + 1) * sizeof(int)));
  if (m->bigram) RB_TRY(zeroed((void**)&s->big_rows, (size_t)rows * sizeof(int)));
  if (m->loop_in.w) RB_TRY(zeroed(&s->cat, (size_t)rows * 2 * m->dp * es));
  RB_TRY(acts_alloc(c, &s->xn2, (size_t)rows * m->dp * es));
  RB_TRY(acts_alloc(c, &s->cq, (size_t)rows * cq * es));
  RB_TRY(acts_alloc(c, (void**)&s->gate, (size_t)rows * heads * sizeof(float)));
  RB_TRY(acts_alloc(c, (void**)&s->part2, s->part_bytes));
  if (m->stack.block != BLOCK_OUTPUT_NORM && m->stack.block != BLOCK_SANDWICH && std::any_of(m->spec.begin(), m->spec.end(), [](const rewb200_layer& L) { return L.shared_ffn > 0; })) {
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
  for (auto* list : {&s->delta_state, &s->delta_conv, &s->lru_state, &s->lru_conv}) list->resize(n, nullptr);
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
    auto recurrent = [&](float** state, int64_t elems, float** conv, const ConvDims& cd) -> int {
      RB_TRY(zeroed((void**)state, (size_t)s->B * elems * sizeof(float)));
      return conv_state_elems(cd) > 0 ? zeroed((void**)conv, (size_t)s->B * conv_state_elems(cd) * sizeof(float)) : REWB200_OK;
    };
    if (has(D, MIX_DELTA)) RB_TRY(recurrent(&s->delta_state[r], (int64_t)D.d.m.heads * D.d.m.dim * gla_state_ld(D.d.m.vdim), &s->delta_conv[r], D.d.conv));
    if (has(D, MIX_LRU)) RB_TRY(recurrent(&s->lru_state[r], (int64_t)D.r.m.blocks * D.r.m.n, &s->lru_conv[r], D.r.conv));
  }
  if (m->bigram) RB_TRY(zeroed((void**)&s->last_ids, (size_t)s->B * sizeof(int)));
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
  s->plan_gqa_small = s->plan_gqa_large = s->plan_delta_small = s->plan_delta_large = s->plan_delta_chunks = s->plan_portions = s->plan_longest = 0;
  if (!uniform) {
    std::vector<int>& h = s->plan_host;
    h.assign(2 * rows, 0);
    std::vector<int2> tiles, chunks, keys;
    std::vector<ExpTile> exps;
    abs_rows = 0;
    int64_t reach = 0;  // the widest window of any layer, 0: everything
    const bool bf = m->cfg.dtype == REWB200_BF16;
    bool exp_ok = bf && c->latent_impl == 0, gqa_ok = bf && c->gqa_impl == 0, gla_ok = bf && c->gla_impl == 0;
    bool has_latent = false, has_gqa = false, has_gla = false, has_delta = false, delta_ok = bf && c->gla_impl == 0;
    int taps = 0;           // of the longest convolution
    for (const LayerDev& D : m->layers) {
      if (has(D, MIX_DELTA)) {
        has_delta = true;
        delta_ok = delta_ok && delta_chunk_ok(D.d.m);
        taps = std::max(taps, D.d.conv.taps);
      }
      if (has(D, MIX_LRU)) taps = std::max(taps, D.r.conv.taps);
      if (D.mixer == MIX_GQA) {
        has_gqa = true;
        gqa_ok = gqa_ok && (gqa_is_mixed(D.g.m) ? gqa_mix_prefill_ok(D.g.m) : gqa_prefill_ok(D.g.m));
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
    std::vector<int2> gla_chunk, tails, delta_chunk;
    std::vector<GlaPortion> delta_small, delta_large, portions;
    for (const StepEntry& e : *o.entries) {
      portions.push_back({e.row0, e.n, e.pos0, e.lane, 0});
      s->plan_longest = std::max(s->plan_longest, e.n);
      if (has_delta) {
        const bool large = delta_ok && e.n >= CHUNK_MIN_ROWS;
        const GlaPortion p = {e.row0, e.n, e.pos0, e.lane, large ? (int)delta_chunk.size() : 0};
        (large ? delta_large : delta_small).push_back(p);
        if (large)
          for (int i = 0; i < delta_chunks(e.n); ++i) delta_chunk.push_back(delta_chunk_rows(p, i));
      }
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
    s->plan_delta_small = (int)delta_small.size();
    s->plan_delta_large = (int)delta_large.size();
    s->plan_delta_chunks = (int)delta_chunk.size();
    s->plan_portions = (int)portions.size();
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
    append(portions.data(), portions.size() * sizeof(GlaPortion));
    append(delta_small.data(), delta_small.size() * sizeof(GlaPortion));
    append(delta_large.data(), delta_large.size() * sizeof(GlaPortion));
    if (h.size() % 2) h.push_back(0);
    append(delta_chunk.data(), delta_chunk.size() * sizeof(int2));
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
  size_t chunk = 0, mix = 0, lse = 0;
  for (const LayerDev& D : m->layers) {
    if (D.mixer == MIX_GLA) chunk = std::max(chunk, gla_chunk_bytes(D.l.m) * s->plan_gla_chunks);
    if (has(D, MIX_DELTA)) chunk = std::max(chunk, delta_chunk_bytes(D.d.m) * s->plan_delta_chunks);
    if (D.mixer != MIX_GQA || !gqa_is_mixed(D.g.m)) continue;
    if (s->plan_gqa_large > 0) lse = std::max(lse, (size_t)rows * D.g.m.heads * sizeof(float));
    if (uniform || s->plan_gqa_small > 0)
      mix = std::max(mix, gqa_mix_bytes(c, D.g.m, m->cfg.dtype, rows, uniform ? rows : s->plan_gqa_small, uniform ? 1 : GQA_TILE_ROWS, (int64_t)s->max_pages * PAGE));
  }
  if (chunk > s->gla_work_bytes) {
    s->gla_work_bytes = 0;
    RB_TRY(regrow(s, &s->gla_work, chunk));
    s->gla_work_bytes = chunk;
  }
  if (lse > s->mix_lse_bytes) {
    s->mix_lse_bytes = 0;
    RB_TRY(regrow(s, &s->mix_lse, lse));
    s->mix_lse_bytes = lse;
  }
  if (mix > s->mix_bytes) {
    s->mix_bytes = 0;
    RB_TRY(regrow(s, &s->mix_work, mix));
    s->mix_bytes = mix;
  }
  int64_t units = 0, stats = 0, qe = 0;
  int64_t g_units = 0, g_stats = 0;
  for (const LayerDev& D : m->layers) {
    if (D.mixer == MIX_GQA && !gqa_is_mixed(D.g.m)) {
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
  const GlaPortion *gla_small = nullptr, *gla_large = nullptr, *portions = nullptr, *delta_small = nullptr, *delta_large = nullptr;
  const int2* delta_chunks = nullptr;
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
  t.portions = t.gla_large + s->plan_gla_large;
  t.delta_small = t.portions + s->plan_portions;
  t.delta_large = t.delta_small + s->plan_delta_small;
  const int* end = reinterpret_cast<const int*>(t.delta_large + s->plan_delta_large);
  t.delta_chunks = reinterpret_cast<const int2*>(end + (end - s->plan_dev) % 2);
  return t;
}

// The mixers read the input projection in s->part (latent attention: s->xn) and leave their output (ahead of the output
// projection) in s->attn.

// ks: slabs of the input projection.
int gqa_mixer(rewb200_session* s, const FwdOpts& o, const StepLists& t, size_t r, int64_t rows, bool in_graph, int ks) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  const int dt = m->cfg.dtype;
  const LayerRun& R = m->runs[r];
  LayerDev& D = m->layers[R.layer];
  GqaDev& G = D.g;
  const int64_t ldq = pad8((int64_t)G.m.heads * G.m.dim);
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
  if (gqa_is_mixed(G.m)) {
    GqaMixArgs ma;
    memset(&ma, 0, sizeof(ma));
    ma.m = G.m;
    ma.map = t.map;
    ma.tiles = t.gqa_small;
    ma.max_tile_rows = t.uniform ? 1 : GQA_TILE_ROWS;
    ma.rows = rows;
    ma.q = s->q;
    ma.ldq = ldq;
    if (G.m.gate_elem) ma.gate = s->part + G.gate_col;
    ma.nsplit = ks;
    ma.split_stride = pa.split_stride;
    ma.ld = pa.ld;
    if (G.m.gate) ma.gate_head = s->gate;
    ma.out = s->attn;
    ma.ldo = D.o.K;
    ma.kc = pa.kc;
    ma.vc = pa.vc;
    if (dt == REWB200_BF16) {
      ma.tm_k = &s->tmK[R.cache];
      ma.tm_v = &s->tmV[R.cache];
    }
    ma.ldk = G.ldk;
    ma.ldv = G.ldv;
    ma.block_table = s->block_table;
    ma.max_pages = s->max_pages;
    ma.dtype = dt;
    ma.work = s->mix_work;
    ma.work_bytes = s->mix_bytes;
    ma.early_kv = in_graph ? 1 : 0;
    ma.status = c->d_status;
    RB_TRY(gqa_mix_launch(c, ma));
    if (!t.uniform && s->plan_gqa_large > 0)
      RB_TRY(gqa_mix_prefill_launch(c, ma, t.gqa_large, s->plan_gqa_large, G.talk ? G.talk_host.data() : nullptr, s->mix_lse));
    if (o.trace) RB_TRY(o.trace->mark(TC_ATTN));
    return REWB200_OK;
  }
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

int gla_mixer(rewb200_session* s, const FwdOpts& o, const StepLists& t, size_t r, int64_t rows, bool in_graph, int ks) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  LayerDev& D = m->layers[m->runs[r].layer];
  GlaDev& A = D.l;
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

// What the two mixers below read of the input projection (columns from `col` on, `ks` slabs) and where their output goes.
struct MixerAt {
  const LinW* in;
  int64_t col, out_col;
  int ks;
};

int delta_mixer(rewb200_session* s, const FwdOpts& o, const StepLists& t, size_t r, int64_t rows, bool in_graph, const MixerAt& at) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  LayerDev& D = m->layers[m->runs[r].layer];
  DeltaDev& A = D.d;
  const size_t es = dtype_size(m->cfg.dtype);
  const int64_t ch = A.conv.channels;
  ConvArgs ca;
  memset(&ca, 0, sizeof(ca));
  ca.m = A.conv;
  ca.partial = s->part + at.col;
  ca.nsplit = at.ks;
  ca.split_stride = rows * at.in->N;
  ca.ld = at.in->N;
  ca.map = t.map;
  ca.capacity = s->max_len;
  ca.out = s->conv;
  ca.ldo = pad8(ch);
  ca.dtype = m->cfg.dtype;
  ca.state = s->delta_conv[r];
  ca.tails = t.tails;
  ca.n_tails = s->plan_tails;
  ca.early = in_graph ? 1 : 0;
  ca.status = c->d_status;
  RB_TRY(conv_launch(c, ca, rows));
  if (o.trace) RB_TRY(o.trace->mark(TC_QKV_POST));
  DeltaArgs da;
  memset(&da, 0, sizeof(da));
  da.m = A.m;
  da.list = t.delta_small;
  da.count = t.uniform ? (int)rows : s->plan_delta_small;
  da.pos0 = s->d_pos;
  da.b0 = o.b0;
  da.x = s->conv;
  da.ldx = ca.ldo;
  da.partial = ca.partial + ch;
  da.nsplit = at.ks;
  da.split_stride = ca.split_stride;
  da.ld = ca.ld;
  da.eps = m->cfg.eps;
  da.state = s->delta_state[r];
  da.ldv = (int)gla_state_ld(A.m.vdim);
  da.out = (char*)s->attn + at.out_col * es;
  da.ldo = D.o.K;
  da.dtype = m->cfg.dtype;
  da.early = in_graph ? 1 : 0;
  da.status = c->d_status;
  RB_TRY(delta_recurrent_launch(c, da));
  if (!t.uniform && s->plan_delta_large > 0) {
    da.list = t.delta_large;
    da.count = s->plan_delta_large;
    da.chunks = t.delta_chunks;
    da.n_chunks = s->plan_delta_chunks;
    da.work = s->gla_work;
    RB_TRY(delta_chunk_launch(c, da));
  }
  if (o.trace) RB_TRY(o.trace->mark(TC_ATTN));
  return REWB200_OK;
}

int lru_mixer(rewb200_session* s, const FwdOpts& o, const StepLists& t, size_t r, int64_t rows, bool in_graph, const MixerAt& at) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  LayerDev& D = m->layers[m->runs[r].layer];
  LruDev& A = D.r;
  const bool bf = m->cfg.dtype == REWB200_BF16;
  const int64_t width = A.conv.channels, ldn = A.m.ldn;
  ConvArgs ca;
  memset(&ca, 0, sizeof(ca));
  ca.m = A.conv;
  ca.partial = s->part + at.col + width;
  ca.nsplit = at.ks;
  ca.split_stride = rows * at.in->N;
  ca.ld = at.in->N;
  ca.map = t.map;
  ca.capacity = s->max_len;
  ca.out = s->conv;
  ca.ldo = ldn;
  ca.group = A.m.n;
  ca.offsets = s->group_rows;
  ca.dtype = m->cfg.dtype;
  ca.state = s->lru_conv[r];
  ca.tails = t.tails;
  ca.n_tails = s->plan_tails;
  ca.early = in_graph ? 1 : 0;
  ca.status = c->d_status;
  RB_TRY(conv_launch(c, ca, rows));
  if (o.trace) RB_TRY(o.trace->mark(TC_QKV_POST));
  // both gates of every block: a stacked matrix per block on the block's channels
  if (bf) {
    RB_TRY(linear_bf16_launch(c, A.plan_gates, (const bf16*)s->conv, ldn, rows * A.m.blocks, EPI_BIAS_F32, 1, s->gate_pre, 2 * ldn, A.gate_bias,
                              s->group_rows, (int)rows));
  } else {
    for (int b = 0; b < A.m.blocks; ++b)
      RB_TRY(gemm_f32_ld_launch(c, (const float*)s->conv + (int64_t)b * rows * ldn, ldn, (const float*)A.gates + (int64_t)b * ldn * 2 * ldn, 2 * ldn,
                                A.gate_bias + (int64_t)b * 2 * ldn, s->gate_pre + (int64_t)b * rows * 2 * ldn, 2 * ldn, rows, ldn, 2 * ldn));
  }
  if (o.trace) RB_TRY(o.trace->mark(TC_GATE_UP));
  LruArgs la;
  memset(&la, 0, sizeof(la));
  la.m = A.m;
  la.list = t.portions;
  la.count = t.uniform ? (int)rows : s->plan_portions;
  la.longest = s->plan_longest;
  la.pos0 = s->d_pos;
  la.b0 = o.b0;
  la.rows = rows;
  la.gates = s->gate_pre;
  la.u = s->conv;
  la.partial = s->part + at.col;
  la.nsplit = at.ks;
  la.split_stride = ca.split_stride;
  la.ld = ca.ld;
  la.state = s->lru_state[r];
  la.out = (char*)s->attn + at.out_col * dtype_size(m->cfg.dtype);
  la.ldo = D.o.K;
  la.dtype = m->cfg.dtype;
  la.early = in_graph ? 1 : 0;
  RB_TRY(lru_launch(c, la));
  if (o.trace) RB_TRY(o.trace->mark(TC_ATTN));
  return REWB200_OK;
}

// A feed-forward, gated SiLU (dense, or the shared expert beside routed ones) or tanh GELU: f32 slabs of the result in `out`,
// without the bias of the down projection.
int dense_ff(rewb200_session* s, const FwdOpts& o, LayerDev& D, const void* x, int64_t rows, float* out, int* ks) {
  rewb200_model* m = s->m;
  const int64_t dp = m->dp;
  if (D.gelu) {
    const bool bf = m->cfg.dtype == REWB200_BF16;
    RB_TRY(run_linear(s, D.gu, x, dp, rows, false, bf ? EPI_GELU_BF16 : EPI_BIAS_F32, bf ? s->h : (void*)s->gu32, D.ffn_local, nullptr));
    if (!bf) RB_TRY(gelu_f32_launch(m->c, s->gu32, (float*)s->h, rows * D.ffn_local));
  } else if (m->cfg.dtype == REWB200_BF16) {
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

// The mixers of run r.  *joined: a second one ran beside the first on the side stream, so what follows has two predecessors.
int mixer(rewb200_session* s, const FwdOpts& o, const StepLists& t, size_t r, int64_t rows, bool in_graph, bool* joined = nullptr) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  LayerDev& D = m->layers[m->runs[r].layer];
  if (D.mixer == MIX_LATENT) return latent_mixer(s, o, t, r, rows, in_graph);
  MixerAt at = {&in_of(D), 0, 0, 1};
  RB_TRY(run_linear(s, *at.in, s->xn, m->dp, rows, true, 0, s->part, at.in->N, &at.ks));
  if (o.trace) RB_TRY(o.trace->mark(TC_QKV));
  auto recurrent = [&](int kind, const MixerAt& p) { return kind == MIX_DELTA ? delta_mixer(s, o, t, r, rows, in_graph, p) : lru_mixer(s, o, t, r, rows, in_graph, p); };
  MixerAt second = at;
  second.col = D.beside_in;
  second.out_col = D.beside_out;
  // small steps are chains of short launches: two chains at a time
  const bool fork = joined && D.beside && D.mixer == MIX_GQA && m->cfg.dtype == REWB200_BF16 && rows <= 64 && c->moe_overlap && !o.trace;
  if (fork)
    RB_TRY(on_side_stream(c, [&]() -> int {
      const bool pdl = c->use_pdl;
      c->use_pdl = false;   // follows an event wait: plain launches
      const int st = recurrent(D.beside, second);
      c->use_pdl = pdl;
      return st;
    }));
  if (D.mixer == MIX_GQA) RB_TRY(gqa_mixer(s, o, t, r, rows, in_graph, at.ks));
  else if (D.mixer == MIX_GLA) RB_TRY(gla_mixer(s, o, t, r, rows, in_graph, at.ks));
  else RB_TRY(recurrent(D.mixer, at));
  if (fork) RB_CUDA(cudaStreamWaitEvent(c->stream, c->ev_join, 0));
  else if (D.beside) RB_TRY(recurrent(D.beside, second));
  if (joined) *joined = fork;
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

// Blocks normed on both sides: x += back1(mixer(norm1(x))), x += back2(ff(norm2(x))).
int sandwich_blocks(rewb200_session* s, const FwdOpts& o, const NormArgs& na, int64_t rows, bool in_graph) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  const int64_t dp = m->dp;
  const size_t es = dtype_size(m->cfg.dtype);
  const StepLists t = step_lists(s, o, rows);
  OutputNormArgs base;
  memset(&base, 0, sizeof(base));
  base.x_res = s->x_res;
  base.split_stride = rows * dp;
  base.eps = m->cfg.eps;
  base.d = dp;
  base.d_mean = na.d_mean;
  base.out = s->xn;
  base.dtype = m->cfg.dtype;
  base.status = c->d_status;
  auto enters = [&](size_t r) { return m->loop_in.w && r < m->runs.size() && m->runs[r].step >= 0; };
  // what the launch that finishes x leaves for run r: its norm (the final one behind the last run), or x itself ahead of a pass
  auto ahead_of = [&](size_t r, OutputNormArgs& a) {
    if (enters(r)) {
      a.out = s->cat;
      a.ldo = 2 * dp;
    } else {
      a.final_gamma = r < m->runs.size() ? m->layers[m->runs[r].layer].ln1g : m->ng;
    }
  };
  if (o.trace) RB_TRY(o.trace->begin(c->stream));
  {
    OutputNormArgs a = base;
    a.embed = na.embed;
    a.embed_scale = m->stack.embed_scale;
    a.ids = na.ids;
    a.vocab = na.vocab;
    if (m->bigram) {
      RB_TRY(bigram_rows_launch(c, na.ids, t.map.row_lane, t.map.row_pos, s->d_pos, o.b0, rows, m->stack.bigram_buckets, m->stack.bigram_mul_prev,
                                m->stack.bigram_mul_cur, m->cfg.vocab, s->last_ids, s->big_rows, c->d_status));
      a.embed2 = m->bigram;
      a.ids2 = s->big_rows;
    }
    if (m->loop_in.w) {
      a.out_x = (char*)s->cat + dp * es;
      a.ldx = 2 * dp;
    }
    ahead_of(0, a);
    RB_TRY(output_norm_launch(c, a, rows));
    if (o.trace) RB_TRY(o.trace->mark(TC_EMBED));
  }
  for (size_t r = 0; r < m->runs.size(); ++r) {
    LayerDev& D = m->layers[m->runs[r].layer];
    if (enters(r)) {
      OutputNormArgs a = base;
      a.nsplit = 1;
      RB_TRY(run_linear(s, m->loop_in, s->cat, 2 * dp, rows, true, 0, s->part, dp, &a.nsplit));
      a.partial = s->part;
      a.replace = 1;
      a.final_gamma = D.ln1g;
      RB_TRY(output_norm_launch(c, a, rows));
      if (o.trace) RB_TRY(o.trace->mark(TC_EMBED));
    }
    bool joined = false;
    RB_TRY(mixer(s, o, t, r, rows, in_graph, &joined));
    OutputNormArgs a = base;
    a.nsplit = 1;
    const bool pdl = c->use_pdl;
    if (joined) c->use_pdl = false;   // two predecessors: a plain dependency
    const int st = run_linear(s, D.o, s->attn, D.o.K, rows, true, 0, s->part, dp, &a.nsplit);
    c->use_pdl = pdl;
    RB_TRY(st);
    if (o.trace) RB_TRY(o.trace->mark(TC_O));
    a.partial = s->part;
    a.gamma = D.back1;
    if (D.ff) a.final_gamma = D.ln2g;
    else ahead_of(r + 1, a);
    RB_TRY(output_norm_launch(c, a, rows));
    if (o.trace) RB_TRY(o.trace->mark(TC_NORM_ATTN));
    if (D.ff) {
      OutputNormArgs b = base;
      b.nsplit = 1;
      RB_TRY(dense_ff(s, o, D, s->xn, rows, s->part, &b.nsplit));
      b.partial = s->part;
      b.bias = D.gelu ? D.down.b : nullptr;
      b.gamma = D.back2;
      ahead_of(r + 1, b);
      RB_TRY(output_norm_launch(c, b, rows));
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
  if (m->stack.block == BLOCK_SANDWICH) return sandwich_blocks(s, o, na, rows, in_graph);
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
