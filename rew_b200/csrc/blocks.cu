// Layered models (rewb200_model_create_layers): weights, caches and the forward of decoders whose layers are described
// one by one.  They share the engine's sessions, lanes, page pool, captured decode step, sampler and lm_head
// (engine.cu); this file has what differs per layer.
//
// A layer is the parallel block x += mixer(norm1(x)) + ff(norm2(x)).  One launch (residual_norm) adds both branches'
// f32 slabs to the residual, adds what a loop adds ahead of a pass, and leaves both norms of the next layer run.
// In small steps the feed-forward branch runs on the slot's second stream beside the mixer.
//
// Device layouts beyond engine.cu's: rows and Linear outputs are padded to multiples of 8 elements (zero weights, zero
// norm weights), so any width can be loaded by TMA; the mixer's four input projections are one matrix; the key and value
// projections of the latent are one matrix; a loop's passes share weights and have a cache each.
#include <cmath>
#include <map>

#include "engine.cuh"

namespace rewb {

namespace {

int64_t pad8(int64_t v) { return (v + 7) / 8 * 8; }

enum Slot : int {
  SL_NORM1, SL_DQ, SL_DQ_NORM, SL_UQ, SL_DKV, SL_DKV_NORM, SL_UK, SL_UV, SL_G, SL_O, SL_NORM2, SL_GATE, SL_UP, SL_DOWN, SL_ROUTER,
  SL_E_GATE, SL_E_UP, SL_E_DOWN, SL_EMBED, SL_STEP, SL_FINAL
};
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
    for (Slot s : {SL_NORM1, SL_DQ, SL_DQ_NORM, SL_UQ, SL_DKV, SL_DKV_NORM, SL_UK, SL_UV}) out->push_back({s, l, -1});
    if (L.out_gate) out->push_back({SL_G, l, -1});
    out->push_back({SL_O, l, -1});
    if (L.ff) out->push_back({SL_NORM2, l, -1});
    if (L.ff == 1)
      for (Slot s : {SL_GATE, SL_UP, SL_DOWN}) out->push_back({s, l, -1});
    if (L.ff == 2) {
      out->push_back({SL_ROUTER, l, -1});
      for (int e = 0; e < L.experts; ++e) {
        if (L.expert_gated) out->push_back({SL_E_GATE, l, e});
        out->push_back({SL_E_UP, l, e});
        out->push_back({SL_E_DOWN, l, e});
      }
    }
  }
  out->push_back({SL_FINAL, -1, -1});
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
  for (int l = 0; l < n; ++l) {
    const rewb200_layer& L = m->spec[l];
    const std::string who = "layer " + std::to_string(l) + ": ";
    RB_REQUIRE(L.mixer == 1, who + "unknown mixer");
    RB_REQUIRE(L.heads > 0 && L.dim > 0 && L.rot_dim >= 0 && L.vdim > 0 && L.q_rank > 0 && L.kv_rank > 0, who + "mixer sizes must be positive");
    RB_REQUIRE(L.rope_dims >= 0 && L.rope_dims % 2 == 0 && L.rope_dims <= L.rot_dim, who + "rotated features must be pairs within rot_dim");
    RB_REQUIRE(L.window >= 0, who + "the window must not be negative");
    RB_REQUIRE(L.ff >= 0 && L.ff <= 2 && (L.ff == 0 || L.ffn > 0), who + "unknown feed-forward");
    RB_REQUIRE(L.ff != 2 || (L.experts > 0 && L.experts <= 256 && L.top_k > 0 && L.top_k <= L.experts),
               who + "experts must be in 1..256 and top in 1..experts");
  }
  const int64_t d = m->cfg.d_model, dp = m->dp = pad8(d);
  m->vp = pad8(m->cfg.vocab);
  RB_TRY(zero_weights(m, &m->embed, (size_t)m->cfg.vocab * dp * es));
  if (st.loop_times > 0) RB_TRY(zero_weights(m, (void**)&m->step_vec, (size_t)st.loop_times * dp * sizeof(float)));
  std::map<std::pair<double, int>, float2*> tables;
  m->layers.resize(n);
  int64_t widest = dp, q_cols = 0, attn_cols = 0;
  for (int l = 0; l < n; ++l) {
    const rewb200_layer& L = m->spec[l];
    LayerDev& D = m->layers[l];
    LatentDev& A = D.a;
    RB_TRY(zero_weights(m, (void**)&D.ln1g, dp * sizeof(float)));
    if (L.ff) RB_TRY(zero_weights(m, (void**)&D.ln2g, dp * sizeof(float)));
    A.m = LatentDims{L.heads, L.dim, L.rot_dim, L.vdim, L.q_rank, L.kv_rank, L.rope_dims, L.window, L.out_gate, L.scale, nullptr, m->cfg.max_seq};
    if (L.rope_dims > 0) {
      float2*& t = tables[{L.rope_base, L.rope_dims}];
      if (!t) RB_TRY(rope_table(m, L.rope_base, L.rope_dims, &t));
      A.m.rope = t;
    }
    RB_TRY(zero_lin(m, &A.in, dp, pad8((int64_t)L.q_rank + L.kv_rank + L.rot_dim + (L.out_gate ? L.heads : 0))));
    RB_TRY(zero_lin(m, &A.uq, pad8(L.q_rank), pad8((int64_t)L.heads * (L.dim + L.rot_dim))));
    RB_TRY(zero_lin(m, &A.ukv, L.kv_rank, pad8((int64_t)L.heads * (L.dim + L.vdim))));
    RB_TRY(zero_weights(m, (void**)&A.q_norm, L.q_rank * sizeof(float)));
    RB_TRY(zero_weights(m, (void**)&A.kv_norm, L.kv_rank * sizeof(float)));
    A.ldc = pad8(L.kv_rank + L.rot_dim);
    RB_TRY(zero_lin(m, &D.o, pad8((int64_t)L.heads * L.vdim), dp));
    widest = std::max(widest, std::max(A.in.N, A.uq.N));
    q_cols = std::max(q_cols, A.uq.N);
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
      X.gated = L.expert_gated != 0;
      X.f = fp;
      const int64_t up = X.gated ? 2 * fp : fp;
      RB_TRY(zero_lin(m, &X.router, dp, pad8(L.experts)));
      RB_TRY(zero_weights(m, &X.gu, (size_t)L.experts * dp * up * es));
      RB_TRY(zero_weights(m, &X.down, (size_t)L.experts * fp * dp * es));
      RB_TRY(zero_weights(m, (void**)&X.gu_b, (size_t)L.experts * up * sizeof(float)));
      RB_TRY(zero_weights(m, (void**)&X.down_b, (size_t)L.experts * dp * sizeof(float)));
      m->max_moe_ffn = std::max(m->max_moe_ffn, fp);
      m->max_experts = std::max<int>(m->max_experts, (int)X.router.N);
      m->max_topk = std::max(m->max_topk, X.top_k);
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
  for (const LayerRun& r : m->runs)
    if (m->layers[r.layer].moe) ++m->n_moe;
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
  LayerDev& D = m->layers[t.layer];
  const rewb200_layer& L = m->spec[t.layer];
  LatentDev& A = D.a;
  const int64_t fp = pad8(L.ffn);
  // gate / up columns: bf16 interleaves groups of 8, f32 concatenates
  const int64_t gran = bf ? 8 : L.ffn, gst = bf ? 16 : L.ffn, uoff = bf ? 8 : fp;
  auto gate_up = [&](void* w, bool up) { return scatter(m, C, 0, 0, R, C, w, true, 2 * fp, gran, gst, up ? uoff : 0); };
  switch (t.slot) {
    case SL_NORM1: return norm(D.ln1g, zc);
    case SL_NORM2: return norm(D.ln2g, zc);
    case SL_DQ_NORM: return norm(A.q_norm, false);
    case SL_DKV_NORM: return norm(A.kv_norm, false);
    case SL_DQ: return cols(A.in.w, A.in.N, 0);
    case SL_DKV: return cols(A.in.w, A.in.N, L.q_rank);
    case SL_G: return cols(A.in.w, A.in.N, (int64_t)L.q_rank + L.kv_rank + L.rot_dim);
    case SL_UQ: return cols(A.uq.w, A.uq.N, 0);
    case SL_UK: return cols(A.ukv.w, A.ukv.N, 0);
    case SL_UV: return cols(A.ukv.w, A.ukv.N, (int64_t)L.heads * L.dim);
    case SL_O: return cols(D.o.w, m->dp, 0);
    case SL_GATE: return gate_up(D.gu.w, false);
    case SL_UP: return gate_up(D.gu.w, true);
    case SL_DOWN: return cols(D.down.w, m->dp, 0);
    case SL_ROUTER: return cols(D.x.router.w, D.x.router.N, 0);
    case SL_E_DOWN: return cols((char*)D.x.down + (size_t)t.expert * fp * m->dp * es, m->dp, 0);
    case SL_E_GATE: return gate_up((char*)D.x.gu + (size_t)t.expert * m->dp * 2 * fp * es, false);
    case SL_E_UP:
      if (D.x.gated) return gate_up((char*)D.x.gu + (size_t)t.expert * m->dp * 2 * fp * es, true);
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
    if (D.ff) RB_TRY(fill_const_launch(c, D.ln2g, REWB200_F32, m->dp, 1.f));
    RB_TRY(fill_const_launch(c, D.a.q_norm, REWB200_F32, D.a.m.q_rank, 1.f));
    RB_TRY(fill_const_launch(c, D.a.kv_norm, REWB200_F32, D.a.m.kv_rank, 1.f));
    for (LinW* w : {&D.a.in, &D.a.uq, &D.a.ukv, &D.o}) RB_TRY(fill(w->w, w->K * w->N));
    if (D.ff == 1)
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
    for (LinW* w : {&D.a.in, &D.a.uq, &D.a.ukv, &D.o}) RB_TRY(plan(*w));
    if (D.ff == 1)
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
  int64_t cq = 0, heads = 0;
  for (const LayerDev& D : m->layers) {
    cq = std::max(cq, D.a.uq.K);
    heads = std::max<int64_t>(heads, D.a.m.heads);
  }
  RB_TRY(acts_alloc(c, &s->xn2, (size_t)rows * m->dp * es));
  RB_TRY(acts_alloc(c, &s->cq, (size_t)rows * cq * es));
  RB_TRY(acts_alloc(c, (void**)&s->gate, (size_t)rows * heads * sizeof(float)));
  RB_TRY(acts_alloc(c, (void**)&s->part2, s->part_bytes));
  if (c->record_layers) RB_TRY(acts_alloc(c, (void**)&s->layer_rec, m->runs.size() * (size_t)rows * m->dp * sizeof(float)));
  // padding columns are multiplied by zero weights, so they must hold finite values from the start
  RB_CUDA(cudaMemsetAsync(s->cq, 0, (size_t)rows * cq * es, c->stream));
  RB_CUDA(cudaMemsetAsync(s->attn, 0, (size_t)rows * m->nq * es, c->stream));
  RB_CUDA(cudaMemsetAsync(s->h, 0, (size_t)rows * std::max<int64_t>(std::max(m->max_ffn, m->max_moe_ffn), 1) * es, c->stream));
  return REWB200_OK;
}

// One cache of latents per layer run.
int layered_session(rewb200_session* s, int64_t n_pages) {
  rewb200_model* m = s->m;
  const size_t es = dtype_size(m->cfg.dtype);
  const size_t n = m->runs.size();
  s->kc.resize(n, nullptr);
  s->tmK.resize(n);
  for (size_t r = 0; r < n; ++r) {
    const int64_t ldc = m->layers[m->runs[r].layer].a.ldc;
    const size_t bytes = (size_t)n_pages * PAGE * ldc * es;
    RB_CUDA(cudaMalloc(&s->kc[r], bytes));
    RB_CUDA(cudaMemsetAsync(s->kc[r], 0, bytes, m->c->stream));
    if (m->cfg.dtype == REWB200_BF16)
      RB_TRY(make_tmap_2d_bf16(&s->tmK[r], s->kc[r], (uint64_t)ldc, (uint64_t)n_pages * PAGE, (uint64_t)ldc * 2, 64, 64));
  }
  return REWB200_OK;
}

namespace {

// Rows of one lane an absorbed-attention tile covers at most.
constexpr int ABS_TILE_ROWS = 8;
// Portions of at least this many tokens attend to keys and values expanded per head.  Expanding costs a Linear over the
// portion's keys, its own and its window's; the absorbed form costs (2 kv_rank + rot_dim) / (dim + rot_dim + vdim) times
// the score and value products of every query, on the slower mma.sync pipe.
constexpr int EXPAND_MIN_ROWS = 64;

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
  // ---- lists of the step: [row lane | row position | absorbed tiles | their chunks | expanded tiles | gathered keys]
  int64_t abs_rows = rows, n_keys = 0;
  s->plan_host.clear();
  s->plan_abs_tiles = s->plan_chunks = s->plan_exp_tiles = s->plan_keys = 0;
  if (!uniform) {
    std::vector<int>& h = s->plan_host;
    h.resize(2 * rows);
    std::vector<int2> tiles, chunks, keys;
    std::vector<ExpTile> exps;
    abs_rows = 0;
    int64_t reach = 0;  // the widest window of any layer, 0: everything
    bool exp_ok = m->cfg.dtype == REWB200_BF16 && c->latent_impl == 0;
    for (const LayerDev& D : m->layers) {
      exp_ok = exp_ok && latent_expanded_ok(D.a.m);
      reach = D.a.m.window == 0 ? INT32_MAX : std::max<int64_t>(reach, D.a.m.window);
    }
    for (const StepEntry& e : *o.entries) {
      for (int i = 0; i < e.n; ++i) {
        h[e.row0 + i] = e.lane;
        h[rows + e.row0 + i] = e.pos0 + i;
      }
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
  int64_t units = 0, stats = 0, qe = 0;
  for (const LayerDev& D : m->layers) {
    const int64_t H = D.a.m.heads;
    const int sp = latent_kv_splits(c, D.a.m, rows, s->max_len);
    units = std::max(units, H * sp * D.a.m.kv_rank);
    stats = std::max(stats, H * sp);
    qe = std::max(qe, H * D.a.ldc);
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

// The layer runs of a layered model over `rows` rows; na carries the residual, the embedding and the ids.  Leaves the
// final norm's output in s->xn.
int layered_blocks(rewb200_session* s, const FwdOpts& o, const NormArgs& na, int64_t rows, bool in_graph) {
  rewb200_model* m = s->m;
  Ctx* c = m->c;
  const int dt = m->cfg.dtype;
  const int64_t dp = m->dp;
  const bool uniform = o.entries == nullptr;
  RowMap map = {nullptr, nullptr, s->d_pos, o.b0, o.S};
  RowTiles abs = {nullptr, (int)rows, 1, 1}, chunks = {nullptr, (int)((rows + kChunkRows - 1) / kChunkRows), 1, 1};
  const ExpTile* exp_tiles = nullptr;
  const int2* key_list = nullptr;
  const bool expand = !uniform && s->plan_exp_tiles > 0;
  if (!uniform) {
    map.row_lane = s->plan_dev;
    map.row_pos = s->plan_dev + rows;
    abs.list = reinterpret_cast<const int2*>(s->plan_dev + 2 * rows);
    abs.count = s->plan_abs_tiles;
    chunks.list = abs.list + abs.count;
    chunks.count = s->plan_chunks;
    exp_tiles = reinterpret_cast<const ExpTile*>(chunks.list + chunks.count);
    key_list = reinterpret_cast<const int2*>(exp_tiles + s->plan_exp_tiles);
  }
  auto ahead_of = [&](size_t r, NormArgs& a) {  // what the norm launch in front of run r adds and writes
    if (r == m->runs.size()) {
      a.gamma = m->ng;
      return;
    }
    const LayerRun& R = m->runs[r];
    const LayerDev& D = m->layers[R.layer];
    a.gamma = D.ln1g;
    if (D.ff) {
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
    LatentDev& A = D.a;
    int ks = 1, ks_o = 1, ks_f = 0;
    const bool fork = D.ff != 0 && dt == REWB200_BF16 && rows <= 64 && c->moe_overlap && !o.trace;
    // ---- feed-forward branch: slabs in part2
    auto ff_branch = [&]() -> int {
      if (D.ff == 0) return REWB200_OK;
      float* const keep = s->part;
      s->part = s->part2;  // scratch and slabs of this branch
      auto body = [&]() -> int {
        if (D.ff == 2) {
          RB_TRY(moe_routed(s, D.x, s->xn2, dp, rows, false, s->part2, moe_seen++, fork));
          ks_f = 1;
          if (o.trace) RB_TRY(o.trace->mark(TC_MOE));
          return REWB200_OK;
        }
        // beside the mixer both Linears are plain launches: a down projection launched early holds shared memory that the
        // mixer's short kernels then wait for (measured, 8B shape: 3.69 instead of 3.53 ms per step at batch 32)
        const bool pdl = c->use_pdl;
        if (fork) c->use_pdl = false;
        auto dense = [&]() -> int {
          if (dt == REWB200_BF16) {
            RB_TRY(run_linear(s, D.gu, s->xn2, dp, rows, false, EPI_SWIGLU_BF16, s->h, D.ffn_local, nullptr));
          } else {
            RB_TRY(run_linear(s, D.gu, s->xn2, dp, rows, false, EPI_BIAS_F32, s->gu32, 2 * D.ffn_local, nullptr));
            RB_TRY(swiglu_rows_f32_launch(c, s->gu32, (float*)s->h, rows, D.ffn_local));
          }
          if (o.trace) RB_TRY(o.trace->mark(TC_GATE_UP));
          return run_linear(s, D.down, s->h, D.ffn_local, rows, true, 0, s->part2, dp, &ks_f);
        };
        const int st = dense();
        c->use_pdl = pdl;
        RB_TRY(st);
        if (o.trace) RB_TRY(o.trace->mark(TC_DOWN));
        return REWB200_OK;
      };
      const int st = body();
      s->part = keep;
      return st;
    };
    if (fork) {
      RB_CUDA(cudaEventRecord(c->ev_fork, c->stream));
      RB_CUDA(cudaStreamWaitEvent(c->side, c->ev_fork, 0));
      cudaStream_t main_stream = c->stream;
      c->stream = c->side;
      const int st = ff_branch();
      c->stream = main_stream;
      RB_TRY(st);
      RB_CUDA(cudaEventRecord(c->ev_join, c->side));
    }
    // ---- mixer
    RB_TRY(run_linear(s, A.in, s->xn, dp, rows, true, 0, s->part, A.in.N, &ks));
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
    pa.map = map;
    pa.cq = s->cq;
    pa.ldcq = A.uq.K;
    pa.gate = s->gate;
    pa.cache = s->kc[r];
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
    aa.map = map;
    aa.tiles = abs;
    aa.chunks = chunks;
    aa.max_tile_rows = uniform ? 1 : ABS_TILE_ROWS;
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
    aa.cache = s->kc[r];
    aa.tm_cache = dt == REWB200_BF16 ? &s->tmK[r] : nullptr;
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
      ea.tiles = exp_tiles;
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
      RB_TRY(latent_gather_launch(c, (const bf16*)s->kc[r], s->block_table, s->max_pages, A.ldc, key_list, (bf16*)s->latx, s->plan_keys));
      RB_TRY(linear_bf16_launch(c, A.ukv.plan, (const bf16*)s->latx, A.ldc, s->plan_keys, EPI_BIAS_BF16, 1, s->kvx, A.ukv.N, nullptr, nullptr, 0));
      RB_TRY(latent_attn_expanded_launch(c, ea));
    }
    if (o.trace) RB_TRY(o.trace->mark(TC_ATTN));
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
    ahead_of(r + 1, a);
    if (a.add_embed) a.embed = m->embed;
    const bool pdl = c->use_pdl;
    if (fork) c->use_pdl = false;  // two predecessors: a plain dependency
    if (s->layer_rec && !uniform) {
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
      a.partial = a.partial2 = nullptr;
      a.nsplit = a.nsplit2 = 0;
    }
    const int st = residual_norm_launch(c, a, rows);
    c->use_pdl = pdl;
    RB_TRY(st);
    if (o.trace) RB_TRY(o.trace->mark(TC_NORM_FFN));
  }
  return REWB200_OK;
}

}  // namespace rewb
