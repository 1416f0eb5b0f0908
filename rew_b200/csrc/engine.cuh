// Model, session and step structures of the engine, shared by engine.cu (grouped-query decoder blocks, sessions,
// generate) and blocks.cu (layered models).
#pragma once
#include <algorithm>
#include <cstring>

#include "common.cuh"
#include "conv.cuh"
#include "delta.cuh"
#include "gla.cuh"
#include "gqa.cuh"
#include "gqa_mix.cuh"
#include "latent.cuh"
#include "lru.cuh"
#include "ptx.cuh"

namespace rewb {

int comm_world(int slot);
int comm_rank(int slot);
int comm_allreduce_sum(Ctx* c, int slot, void* ptr, int64_t n, int dtype);
int comm_allgather_bytes(Ctx* c, int slot, const void* send, void* recv, size_t bytes_per_rank);
int comm_check_async(int slot);
int slab_sum_launch(Ctx* c, float* part, int nsplit, int64_t slab_elems);
int epoch_bump_launch(Ctx* c, int* epoch, int by);
int comm_alltoall_bytes(Ctx* c, int slot, const void* send, void* recv, size_t bytes_per_peer);
int comm_alltoallv_rows(Ctx* c, int slot, const void* send, void* recv, size_t peer_stride_bytes, size_t row_bytes,
                        const int* send_rows, const int* recv_rows);
int moe_route_launch(Ctx* c, const float* logits, int64_t N, int E, int k, float* topw, int* topi);
int moe_route_slabs_launch(Ctx* c, const float* logits, int nsplit, int64_t split_stride, const float* bias, int64_t N, int E,
                           int64_t ld, int k, int renorm, float scale, float* shared_gate, float* topw, int* topi, int* zero, int n_zero);
int moe_group_local_launch(Ctx* c, const void* x, int dtype, const int* topi, int64_t tokens, int k, int64_t d, int n_experts,
                           int* offsets, void* xs, int* pair_pos);
int moe_reset_launch(Ctx* c, int* cursor, int n_cursor, int* count, int n_count, int* meta, int n_meta);
int moe_dispatch_launch(Ctx* c, const void* x, int dtype, const int* topi, int64_t tokens, int k, int64_t d,
                        int experts_per_rank, int capacity, int* cursor, void* send_x, int* send_meta, int* pair_slot);
int moe_group_launch(Ctx* c, const void* recv_x, int dtype, const int* recv_meta, int n_slots, int64_t d, int n_experts,
                     int* count, int* offsets, int* cursor2, void* xs, int* slot_pos);
int moe_return_launch(Ctx* c, const float* ys, const int* slot_pos, int n_slots, int64_t d, float* ret);
int moe_combine_launch(Ctx* c, const float* back, const int* pair_slot, const float* topw, int64_t tokens, int k, int64_t d,
                       float* out, int accumulate);
int moe_dispatch_peer_launch(Ctx* c, const void* x, int dtype, const int* topi, int64_t tokens, int k, int64_t d,
                             int experts_per_rank, int capacity, int* cursor, int* pair_slot, const A2aArgs& a);
int moe_group_peer_launch(Ctx* c, int dtype, int n_slots, int capacity, int64_t d, int n_experts, int* count, int* offsets,
                          int* cursor2, void* xs, int* slot_pos, const A2aArgs& a);
int moe_return_peer_launch(Ctx* c, const float* ys, const int* slot_pos, int n_slots, int capacity, int64_t d, const A2aArgs& a);
int moe_combine_peer_launch(Ctx* c, const int* pair_slot, const float* topw, int64_t tokens, int k, int64_t d, float* out,
                            int accumulate, const A2aArgs& a);
int sample_launch(Ctx* c, const float* logits, float* work, int64_t B, int64_t V, int* hist, int* hist_len, int hist_cap,
                  uint32_t* keys, int* steps, int* next, float* logprob, int logprob_cap, float temperature, int top_k,
                  float top_p, float min_p, float rep_penalty, int do_sample, const int* active);
int argmax_partial_launch(Ctx* c, const float* logits, int64_t rows, int64_t V, int idx_offset, int nchunks, float* pv, int* pi);
int argmax_gathered_launch(Ctx* c, const void* gathered, int world, int64_t rows, int nchunks, int* out);

constexpr int PAGE = 64;

struct LinW {
  void* w = nullptr;   // [K,N] model dtype (for a quantised Linear: the shared dequantisation scratch)
  float* b = nullptr;  // [N]
  int64_t K = 0, N = 0;
  LinearBf16Plan plan;
  bool quant = false;  // weight held as NF4 codes
  Nf4W nf4;
  ColMap cm = {1, 1, 1, 0};  // logical column (the reference's [in,out]) -> device column of `w`
};

// Routed experts of one MoE layer held by this rank (src/rew/models/deepseek.nim:36-52).
struct MoeDev {
  LinW router;                 // gate: [d, n_routed] (layered models: columns padded to a multiple of 8)
  void* gu = nullptr;          // [E_l][d][2f]  gate|up per expert (bf16: interleaved in groups of 8); ungated: up [E_l][d][f]
  float* gu_b = nullptr;       // [E_l][2f]
  void* down = nullptr;        // [E_l][f][d]
  float* down_b = nullptr;     // [E_l][d]
  LinearBf16Plan plan_gu, plan_down;
  int E_l = 0;
  int E = 0;                   // routed experts of the layer, all ranks
  int top_k = 0;
  int renorm = 1;              // routing weights divided by their sum
  float scale = 1.f;           // ... times this
  bool shared_gate = false;    // column E of the router projects the gate of the shared expert
  bool gated = true;           // SwiGLU experts; false: W_down relu(W_up x)^2
  int64_t f = 0;
  std::vector<float> shared_down_bias;  // sum of the shared experts' down biases (uploaded at finalize)
};

// Latent attention of one layer (latent.cuh).
struct LatentDev {
  LatentDims m = {};
  LinW in;                     // [d, q_rank | kv_rank | rot_dim | heads]: query latent, key/value latent, shared key part (own_kv), gate
  LinW uq;                     // [q_rank, heads * (dim + rot_dim)]
  LinW ukv;                    // [kv_rank, heads * dim | heads * vdim]
  float *q_norm = nullptr, *kv_norm = nullptr, *sink = nullptr;
  int64_t ldc = 0;             // elements of a cache row: kv_rank + rot_dim, padded
};

// Grouped-query attention of one layer of a layered model (gqa.cuh).
struct GqaDev {
  GqaDims m = {};
  LinW in;                     // [d, heads * dim | kv_heads * dim | kv_heads * vdim | heads]: queries, keys, values (unless v_from_k), gate
  float *q_norm = nullptr, *k_norm = nullptr, *bias = nullptr, *sink = nullptr, *conv = nullptr, *in_bias = nullptr, *talk = nullptr;
  int64_t gate_col = 0;        // of the gate in `in`
  std::vector<float> talk_host;   // the matrix that mixes the heads, read back when the model is finished
  int64_t ldk = 0, ldv = 0;    // elements of a cached key / value row, padded
};

// Gated linear attention of one layer (gla.cuh).
struct GlaDev {
  GlaDims m = {};
  LinW in;                     // [d, heads * dim | heads * dim | heads * vdim | heads * vdim | rank]: q, k, v, gate, decay features
  float *a2 = nullptr, *a2_b = nullptr, *norm = nullptr;
};

// Gated delta rule of one layer (delta.cuh).
struct DeltaDev {
  DeltaDims m = {};
  ConvDims conv = {};          // of queries, keys and values
  LinW in;                     // [d, kv_heads * dim | kv_heads * dim | heads * vdim | heads * vdim | heads | heads]: q, k, v, gate, step, decay
  float *w = nullptr, *rate = nullptr, *dt_bias = nullptr, *norm = nullptr;
};

// Linear recurrent unit of one layer (lru.cuh).
struct LruDev {
  LruDims m = {};
  ConvDims conv = {};
  LinW in;                     // [d, width | width]: output branch, recurrent branch
  void* gates = nullptr;       // [blocks][ldn][2 ldn]: both gates of a block
  LinearBf16Plan plan_gates;
  float *w = nullptr, *x_bias = nullptr, *conv_bias = nullptr, *y_bias = nullptr, *gate_bias = nullptr, *decay = nullptr;
};

struct LayerDev {
  float *ln1g = nullptr, *ln1b = nullptr, *ln2g = nullptr, *ln2b = nullptr;
  LinW qkv, o, gu, down;       // for a MoE layer gu/down are the fused SHARED experts (width n_shared * moe_ffn)
  int64_t ffn_local = 0;
  bool moe = false;
  MoeDev x;
  int mixer = 0;               // layered models: rewb200_layer::mixer, and what it has
  LatentDev a;
  GqaDev g;
  GlaDev l;
  DeltaDev d;
  LruDev r;
  int beside = 0;              // mixer of the second one on the same input, and the first of its columns in the first one's
  int64_t beside_in = 0, beside_out = 0;   // input projection and of its rows in `o`
  float *back1 = nullptr, *back2 = nullptr;   // norms of the sublayers' outputs
  int ff = 0;                  // layered models: rewb200_layer::ff
  bool gelu = false;           // dense feed-forward W_down gelu(W_up x)
};

// One execution of a layer of a layered model; a layer inside the loop runs once per pass, each with its own cache.
struct LayerRun {
  int layer = 0;
  bool add_embed = false;      // the embedding output is added to the residual ahead of this run
  int step = -1;               // row of the model's step vectors added ahead of this run
  int cache = -1;              // run whose cache this one reads (its own unless the layer shares another's latents or keys and values)
};

}  // namespace rewb

using namespace rewb;

struct rewb200_model {
  Ctx* c = nullptr;
  int slot = 0;
  rewb200_config cfg;
  int nh_l = 0, kvh_l = 0;      // local heads under tensor parallelism
  int64_t vocab_l = 0;          // local slice of the vocabulary (lm_head is vocab-parallel)
  int64_t nq = 0, nkv = 0, nqkv = 0;
  void* embed = nullptr;
  std::vector<LayerDev> layers;
  float *ng = nullptr, *nb = nullptr;
  LinW lm;
  float *cosT = nullptr, *sinT = nullptr;
  float* stage = nullptr;       // f32 upload staging
  size_t stage_bytes = 0;
  bool finalized = false;
  // layered models (rewb200_model_create_layers)
  bool layered = false;
  std::vector<rewb200_layer> spec;
  rewb200_stack stack = {};
  std::vector<LayerRun> runs;
  float* step_vec = nullptr;    // [loop_times][dp]
  void* bigram = nullptr;       // [bigram_buckets + 1][dp]
  LinW loop_in;                 // [2 dp, dp]
  int64_t dp = 0;               // row stride of the residual stream: d_model, padded to a multiple of 8 (layered)
  int64_t vp = 0;               // columns of the lm_head matrix: the vocabulary, padded
  int max_topk = 0, max_experts = 0, n_moe = 0;   // n_moe: MoE layer runs of a step
  int64_t max_ffn = 0, max_moe_ffn = 0;
  int n_cache() const { return layered ? (int)runs.size() : cfg.n_layers; }
  int64_t weight_bytes = 0;
  std::vector<void*> allocs;
};

struct rewb200_session {
  rewb200_model* m = nullptr;
  int B = 0, max_len = 0, max_pages = 0;
  std::vector<void*> kc, vc;           // per layer
  std::vector<CUtensorMap> tmK, tmV;   // per layer (bf16)
  std::vector<float*> state;           // layered models: recurrent or convolution state per layer run [B][..] f32, or nullptr
  std::vector<float*> delta_state, delta_conv, lru_state, lru_conv;  // recurrent and convolution states of the mixers that have both
  int* last_ids = nullptr;             // the last id of every lane (bigram tables)
  int* block_table = nullptr;
  int *d_pos = nullptr, *d_ids = nullptr, *d_next = nullptr, *d_out = nullptr, *d_step = nullptr;
  int out_capacity = 0;
  int32_t* h_ids = nullptr;            // pinned
  // activations, sized for `rows_cap` rows
  int64_t rows_cap = 0;
  float* x_res = nullptr;
  void* xn = nullptr;
  void* q = nullptr;
  void* attn = nullptr;
  void* h = nullptr;
  float* part = nullptr;               // split-K partials (largest user)
  size_t part_bytes = 0;
  float* gu32 = nullptr;               // f32 path: gate|up GEMM output
  float* logits = nullptr;             // [B or rows][V]
  int64_t logits_rows = 0;
  float* attn_scratch = nullptr;
  size_t attn_scratch_bytes = 0;
  void* argmax_scratch = nullptr;      // [B][64] (value, index) partials
  void* gather_scratch = nullptr;      // tensor parallel: all-gathered argmax partials / logits
  size_t gather_bytes = 0;
  // MoE scratch, sized for rows_cap tokens (capacity = tokens * top_k slots per peer)
  float* moe_logits = nullptr;
  float* moe_topw = nullptr;
  int* moe_topi = nullptr;
  int* moe_ints = nullptr;             // cursor | count | offsets | cursor2 | send_meta | recv_meta | pair_slot | slot_pos | recv counts
  size_t moe_ints_n = 0;
  void *moe_send = nullptr, *moe_recv = nullptr, *moe_xs = nullptr, *moe_hs = nullptr;
  float *moe_ys = nullptr, *moe_ret = nullptr, *moe_back = nullptr, *moe_tmp = nullptr;
  int* route_rec = nullptr;            // option record_routing: every MoE layer's top-k expert ids of the last forward, [n_moe][rows_cap][max_topk]
  // layered models
  void* xn2 = nullptr;                 // the second norm of the residual (input of the feed-forward)
  void* cq = nullptr;                  // normed query latents
  float* gate = nullptr;               // output gates [rows][heads]
  float* part2 = nullptr;              // slabs and scratch of the feed-forward branch
  float* part3 = nullptr;              // ... of a shared expert beside routed ones in a parallel block
  float* shared_gate = nullptr;        // its gate [rows]
  void* qeff = nullptr;                // absorbed queries, latent outputs and their row statistics (absorbed rows of a step)
  float* olat = nullptr;
  float2* ml = nullptr;
  int64_t abs_units = 0, abs_stats = 0, abs_rows = 0; // capacity of olat, ml and qeff
  float* gqa_part = nullptr;           // partial outputs of split attention and their row statistics
  float2* gqa_ml = nullptr;
  int64_t gqa_units = 0, gqa_stats = 0;
  void *kvx = nullptr, *latx = nullptr;  // keys / values expanded per head, and the gathered cache rows they come from
  int64_t kvx_rows = 0;
  void* cat = nullptr;                 // rows [x | embeddings] that open a pass of a loop
  void* conv = nullptr;                // what leaves a convolution
  float* gate_pre = nullptr;           // gates of a linear recurrent unit ahead of their sigmoids
  int* group_rows = nullptr;           // first row of every block of them
  int* big_rows = nullptr;             // rows of the bigram table
  float* mix_work = nullptr;           // scores of attention with mixed heads
  size_t mix_bytes = 0;
  float* mix_lse = nullptr;            // its softmax denominators in large portions
  size_t mix_lse_bytes = 0;
  float* layer_rec = nullptr;          // option record_layers: [runs][rows_cap][d]
  int64_t layer_rows = 0;
  void* xg = nullptr;                  // rows of xn gathered for the lm_head
  int64_t xg_rows = 0;
  float* logits_pad = nullptr;         // lm_head output with padded columns (vocabularies that are no multiple of 8)
  int* plan_dev = nullptr;             // row maps, tile lists and gather lists of a step that is no captured decode
  size_t plan_cap = 0;
  std::vector<int> plan_host;
  int plan_abs_tiles = 0, plan_chunks = 0, plan_exp_tiles = 0, plan_keys = 0, plan_tails = 0;
  int plan_gqa_small = 0, plan_gqa_large = 0, plan_gla_small = 0, plan_gla_large = 0, plan_gla_chunks = 0;
  int plan_delta_small = 0, plan_delta_large = 0, plan_delta_chunks = 0, plan_portions = 0, plan_longest = 0;
  uint8_t* gla_work = nullptr;         // blocks of the chunks of gated linear attention or of the delta rule
  size_t gla_work_bytes = 0;
  int* feed_dev = nullptr;             // ids and row lists of a rewb200_lanes_feed step
  size_t feed_cap = 0;
  int64_t route_rows = 0;              // rows of the forward recorded last
  cudaGraphExec_t graph = nullptr;
  cudaEvent_t ev0 = nullptr, ev1 = nullptr;
  float prefill_ms = 0.f, decode_ms = 0.f;
  int host_pos = 0;                    // tokens so far (all sequences advance together)
  int graph_kernels = 0;               // kernels in one captured decode step
  int graph_epoch = -1;                // option epoch the graph was captured under
  // GenerationConfig sampling (generate.nim:12-58); off = greedy argmax
  bool samp_on = false;
  float samp_temperature = 1.f, samp_top_p = 1.f, samp_min_p = 0.f, samp_rep = 1.f;
  int samp_top_k = 0, samp_do_sample = 0;
  std::vector<uint64_t> samp_seeds;    // one per sequence; keys restart from these on reset
  int *samp_hist = nullptr, *samp_hist_len = nullptr, *samp_steps = nullptr;  // [B][max_len], [B], [B]
  uint32_t* samp_keys = nullptr;       // [B][2]
  float *samp_work = nullptr, *samp_logprob = nullptr;  // [B][V], [B][max_len]
  // Paged lanes (continuous batching): a shared pool of KV pages handed out on demand
  bool paged = false;
  int num_blocks = 0;                  // pages in the pool; page 0 is the scratch page of idle lanes
  std::vector<int> free_blocks;        // as PagedKvCache.freeBlocks (generate.nim:75,86-88)
  std::vector<int> lane_len;           // tokens in the cache per lane
  std::vector<char> lane_active;
  std::vector<std::vector<int>> lane_pages;
  int* d_active = nullptr;             // [B] or nullptr (every lane active)
  int* d_ids_prefill = nullptr;        // ids of a single-lane prefill
};

namespace rewb {

// Per-category device times of one forward (REW_B200_TRACE-style measurement aid): an event after the
// launches of each category, elapsed times summed per category after a synchronisation.  Events between
// kernels switch programmatic dependent launch off at those points, so the sum exceeds the untraced step;
// the split is what it is for.
enum TraceCat : int { TC_EMBED = 0, TC_QKV, TC_QKV_POST, TC_ATTN, TC_O, TC_NORM_ATTN, TC_GATE_UP, TC_DOWN, TC_MOE, TC_NORM_FFN, TC_HEAD, TC_COUNT };
struct Trace {
  std::vector<cudaEvent_t> ev;
  std::vector<int> cat;
  cudaStream_t st = nullptr;
  int begin(cudaStream_t s) {
    st = s;
    return mark(-1);
  }
  int mark(int c) {
    cudaEvent_t e;
    RB_CUDA(cudaEventCreate(&e));
    RB_CUDA(cudaEventRecord(e, st));
    ev.push_back(e);
    cat.push_back(c);
    return REWB200_OK;
  }
  int finish(float* ms) {  // ms[TC_COUNT]
    for (int i = 0; i < TC_COUNT; ++i) ms[i] = 0.f;
    RB_CUDA(cudaStreamSynchronize(st));
    for (size_t i = 1; i < ev.size(); ++i) {
      float t = 0.f;
      RB_CUDA(cudaEventElapsedTime(&t, ev[i - 1], ev[i]));
      if (cat[i] >= 0 && cat[i] < TC_COUNT) ms[cat[i]] += t;
    }
    return REWB200_OK;
  }
  ~Trace() {
    for (cudaEvent_t e : ev) cudaEventDestroy(e);
  }
};

// A portion of a step: rows row0 .. row0 + n - 1 are the tokens at positions pos0 .. of `lane`.
struct StepEntry {
  int lane, row0, n, pos0;
};

struct FwdOpts {
  Trace* trace = nullptr;     // when set, an event follows every category of launches
  int S = 1;
  int rope_shift = 0;
  int causal = 1;
  bool all_logits = false;  // lm_head on every row instead of the last position
  bool from_device_ids = false;
  // Lanes [b0, b0 + nb) of the session only (nb < 0: all).  The per-lane arrays (positions, block table,
  // next ids, logits rows, sampling state) are indexed from b0; ids_src overrides where the nb*S input
  // ids are read, so that a single-lane prefill does not disturb the other lanes' pending tokens.
  int b0 = 0, nb = -1;
  const int* ids_src = nullptr;
  bool record_out = true;    // append the new ids to the session's [step][B] output buffer
  // Steps of unequal portions (rewb200_lanes_feed) and layered steps of more than one token: the portions, in row order
  const std::vector<StepEntry>* entries = nullptr;
  // lm_head on these rows (device list) instead of the last row of every lane: n_want rows whose logits are only
  // read back, then the last rows of lanes [b0, b0 + nb) if `sample`
  const int* out_rows = nullptr;
  int n_want = 0;
  bool sample = true;
  const int* sample_active = nullptr;  // overrides the session's active flags for sampling and advance
  int advance = -1;                    // tokens every active lane moves on (-1: S)
};

// ---- engine.cu
int samp_restart(rewb200_session* s);
int dev_alloc(rewb200_model* m, void** p, size_t bytes);
int alloc_lin(rewb200_model* m, LinW* w, int64_t K, int64_t N);
int upload_stage(rewb200_model* m, const float* host, int64_t numel);
int scatter(rewb200_model* m, int64_t src_ld, int64_t row0, int64_t col0, int64_t rows, int64_t cols, void* dst,
            bool dst_model_dtype, int64_t ldd, int64_t gran, int64_t gstride, int64_t off);
int acts_alloc(Ctx* c, void** p, size_t bytes);
int run_linear(rewb200_session* s, const LinW& w, const void* x, int64_t ldx, int64_t rows, bool partial, int epi,
               void* out, int64_t ldo, int* ksplit_out, const QkvPostArgs* fuse_qkv = nullptr, bool* fused = nullptr);
int swiglu_rows_f32_launch(Ctx* c, const float* gu, float* out, int64_t rows, int64_t f);
int gelu_f32_launch(Ctx* c, const float* x, float* out, int64_t n);
// Routed experts of one MoE layer for the normalised rows x [rows][d]: router, top-k, expert Linears, weighted sum
// into `out` (nullptr: slab 0 of s->part).
int moe_routed(rewb200_session* s, MoeDev& X, const void* x, int64_t d, int64_t rows, bool accumulate, float* out = nullptr,
               int moe_index = 0, bool first_plain = false);

// ---- blocks.cu: layered models
int layered_create(rewb200_model* m, const rewb200_layer* layers, const rewb200_stack* stack);
int64_t layered_tensor_count(const rewb200_model* m);
int layered_tensor_shape(const rewb200_model* m, int64_t index, int* ndims, int64_t* shape);
int layered_set_tensor(rewb200_model* m, int64_t index, const float* host, int64_t numel);
int layered_init_random(rewb200_model* m, uint64_t seed, float std);
int layered_plans(rewb200_model* m);
int layered_acts(rewb200_session* s, int64_t rows);
int layered_session(rewb200_session* s, int64_t n_pages);
// Host-side preparation of a step: plan upload and scratch growth (never inside a capture).
int layered_prepare(rewb200_session* s, const FwdOpts& o, int64_t rows);
int layered_blocks(rewb200_session* s, const FwdOpts& o, const NormArgs& na, int64_t rows, bool in_graph);

}  // namespace rewb
