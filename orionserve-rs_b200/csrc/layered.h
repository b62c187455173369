// Layer-list models: decoders whose layers are listed one by one, each with its own token mixer, feed-forward and sizes.
// Four kinds of block:
//   parallel  h = norm(x); mixer and feed-forward each read h plus a short causal convolution of h; both results are added to
//             x. They write their activations next to each other into one buffer and their output matrices are stored side by
//             side along k, so the two sublayers end in a single projection whose accumulator adds them.
//   sandwich  x += m * norm(mixer(norm(x))), then x += m * norm(feed-forward(norm(x))): one kernel folds a sublayer's output
//             projection, normalises it, adds it and normalises the sum for the next sublayer.
//   prenorm   x += m * mixer(norm(x)), then x += m * feed-forward(norm(x)).
//   gated post-norm  x += m * norm(g * mixer(x)), then x += m * norm(g' * feed-forward(x)): the gates are projections of x, stored
//             below the matrix that the sublayer applies to x first (the mixer's joint projection, the router), so they cost no
//             launch of their own; the kernel that normalises and adds a sublayer's output reads them from that product.
// A run of layers may be passed through several times (prenorm blocks): the passes share the weights, and each has caches and states
// of its own, so a pass is simply a further layer of the sequence of layer runs that points to the same weights.
// What a sequence carries from step to step is the paged cache of its attention layers (latents, or keys and values; where the
// embedding looks at the previous token, also the tokens themselves) and, in a state slot, the recurrences' states and the
// convolutions' last inputs.
#pragma once

#include <string>

#include "step_model.h"

namespace orion {

template <typename T>
class LayeredModel final : public StepModel<T> {
  using Base = StepModel<T>;
  using Base::alloc;
  using Base::embed_, Base::lm_head_, Base::finalized_, Base::hidden_, Base::partial_, Base::normed_, Base::tail_, Base::partial_floats_,
      Base::d_meta_, Base::meta_, Base::stream_, Base::ordinal_, Base::prof_on_, Base::only_mask_, Base::stage_f32_, Base::stage_f32_cap_,
      Base::upload_slice, Base::ensure_stage, Base::fill_random, Base::set_constant, Base::timed, Base::run_head, Base::plan_for;

 public:
  LayeredModel(OrionBackend *backend, const OrionLayeredDesc &d) : Base(backend), d_(d), specs_(d.layers, d.layers + d.num_layers) {
    d_.layers = specs_.data();
    desc_ = OrionModelDesc{};
    desc_.hidden_size = d.hidden_size, desc_.num_layers = d.num_layers, desc_.vocab_size = d.vocab_size;
    desc_.max_position_embeddings = d.max_position_embeddings, desc_.rms_norm_eps = (float)d.norm_eps, desc_.tied_lm_head = !d.untied_lm_head;
    desc_.num_blocks = d.num_blocks, desc_.block_size = d.block_size, desc_.compute_dtype = d.compute_dtype;
    desc_.max_batch_tokens = d.max_batch_tokens, desc_.max_batch_sequences = d.max_batch_sequences, desc_.tp_world = 1;
  }

  ~LayeredModel() override {
    cudaSetDevice(ordinal_);
    if (stream_) cudaStreamSynchronize(stream_);
    for (void *p : {(void *)ext_latents_, (void *)ext_rot_, (void *)ext_kv_, gla_scratch_})
      if (p) cudaFree(p);
  }

  int init();
  int load_tensor(const char *name, int dtype, const uint64_t *shape, int ndim, const void *data) override;
  bool uses_tensor(const char *name) const override {
    Place p;
    return place(name, &p);
  }
  int init_random(uint64_t seed, float std) override;
  int finalize() override;
  int fill_kv_random(uint64_t seed, float std) override;
  int read_kv(float *out, uint64_t capacity) override;
  uint32_t num_state_slots() const override { return has_state() ? d_.num_state_slots : 0; }
  bool logical_positions() const override { return true; }
  uint64_t sequence_limit() const override { return d_.learned_positions; }
  float logit_softcap() const override { return (float)d_.logit_softcap; }
  const OrionModelDesc &desc() const override { return desc_; }

 private:
  struct Layer {
    OrionLayerDesc d;
    LatentShape ls{};
    AttnInputs in{};   // attention: the joint projection, cache and form
    KvLayout kv{};
    AttnForm form{};
    bool tuned = false;  // attention: the sizes the tensor-core kernels take
    GlaShape gla{};
    // what joins the stream ahead of this run: a vector (may be null), and what entered the model's first layer
    const float *shift = nullptr;
    bool restart = false;
    MoeShape moe{};      // experts = 0: dense feed-forward or none
    // joint mixer projection's columns, mixer output, columns of the feed-forward's activations and of the output projection
    uint32_t mix_in = 0, mix_out = 0, ff_at = 0, cat = 0, ff_ld = 0;
    // gated post-norm block: first column of a sublayer's gate in the mixer's joint projection, and in the router's
    uint32_t gate_at = 0, ff_gate_at = 0;
    float *norm = nullptr, *mix_bias = nullptr, *latent_norm = nullptr;
    float *norm_post = nullptr, *norm2 = nullptr, *norm2_post = nullptr;  // sandwich block
    float *gate_bias = nullptr, *ff_gate_bias = nullptr;                   // gated post-norm block
    T *w_ff_gate = nullptr;                                                // its gate of a dense feed-forward
    float *q_gain = nullptr, *dist_mult = nullptr, *dist_rate = nullptr;  // keys as values: gains of queries times those of keys
    float *q_norm = nullptr, *k_norm = nullptr, *sinks = nullptr, *up_bias = nullptr, *down_bias = nullptr;
    T *conv1 = nullptr, *conv2 = nullptr, *w_mix = nullptr, *w_up = nullptr, *w_out = nullptr, *w_down = nullptr, *w_uk = nullptr, *w_uv = nullptr;
    T *w_decay = nullptr;        // gla: [heads * dim][rank], its bias in mix_bias
    float *out_norm = nullptr, *correction = nullptr;
    T *w_router = nullptr, *e_up = nullptr, *e_down = nullptr, *s_up = nullptr, *s_down = nullptr;
    T *conv_state = nullptr;     // [2 * slots][taps - 1][hidden]
    float *rec_state = nullptr;  // [2 * slots][width, or a matrix per head]
    T *cache = nullptr;          // latents: [blocks][block_size][row_stride]; keys and values: a KvLayout of one layer
    const float *rope_cos = nullptr, *rope_sin = nullptr;
    bool latent() const { return d.mixer == ORION_MIXER_LATENT_ATTENTION; }
    bool attention() const { return d.mixer == ORION_MIXER_ATTENTION; }
    bool linear() const { return d.mixer == ORION_MIXER_GLA; }
    bool gated_ffn() const { return d.activation == ORION_ACT_GEGLU_TANH; }
    bool has_ffn() const { return d.ffn_dim > 0; }
    size_t cache_elems() const { return latent() ? (size_t)ls.block_size * ls.row_stride : (attention() ? kv.num_kv_heads * kv.chunk_elems() : 0); }
  };
  // Where a checkpoint tensor goes: rows x cols of it into a matrix of row stride `ld` (dst) or a vector (vec).
  struct Place {
    T *dst = nullptr;
    float *vec = nullptr;
    uint64_t rows = 0, cols = 0, ld = 0;
    bool matrix = true, transposed = false;  // transposed: kept as [cols][rows]
    float fill = 1.0f;                       // a vector's value in a randomly initialised model
    uint64_t copies = 0;                     // not 0: the tensor is one number, kept as a vector of this size
  };
  bool place(const std::string &name, Place *p) const;
  std::vector<std::string> tensor_names() const;
  int check_layer(uint32_t i) const;
  int init_layer(Layer &L);
  int init_memory(Layer &L);  // what a layer run keeps of its sequences
  int init_rope(Layer &L);
  int init_query_factors(Layer &L);
  int init_buffers();
  bool sandwich() const { return d_.block == ORION_BLOCK_SANDWICH; }
  bool parallel() const { return d_.block == ORION_BLOCK_PARALLEL; }
  bool gated_postnorm() const { return d_.block == ORION_BLOCK_GATED_POSTNORM; }
  bool has_state() const {
    if (parallel()) return true;
    for (const OrionLayerDesc &s : specs_)
      if (s.mixer == ORION_MIXER_MIN_GRU || s.mixer == ORION_MIXER_GLA) return true;
    return false;
  }
  template <typename U>
  int zeroed(U **p, size_t n) {
    ORION_TRY(alloc(p, n));
    ORION_CUDA_CHECK("clear buffer", cudaMemsetAsync(*p, 0, (n ? n : 1) * sizeof(U), stream_));
    return ORION_OK;
  }

  int run_step_body(bool want_argmax, int part) override;
  int run_parallel_layers();
  int run_sandwich_layers();
  int run_prenorm_layers();
  int run_gated_postnorm_layers();
  bool graph_eligible() const override {
    return g_step_graph && DTypeOf<T>::is_bf16 && meta_.decode && !meta_.zero_count && !prof_on_ && only_mask_ == 0 &&
           (!parallel() || residual_norm_conv_supported(d_.hidden_size, d_.conv_taps));
  }
  void graph_plan(uint32_t *splits, uint32_t *blocks_per_split) const override {
    // the context splits of every attention layer, folded into one word
    uint32_t h = 2166136261u;
    for (const Layer &L : layers_)
      if (tuned(L) || L.tuned) h = (h ^ context_splits(L, meta_.rows)) * 16777619u;
    *splits = h, *blocks_per_split = 0;
  }
  int check_batch(const BatchView &b) override;
  // [first row of each sequence, S + 1][state copy to read, S][to write, S][rows that decode, kFewRows * S]
  size_t extra_words(uint64_t seqs) const override { return (3 + kFewRows) * seqs + 1; }
  void fill_extra(const BatchView &b, uint32_t *w) override;
  void step_done(const BatchView &b) override;
  int poll_errors() override;
  // Sequences with at most this many rows in a batch decode: each row reads the cache by itself.
  static constexpr uint32_t kFewRows = 8;
  size_t tile_words(uint64_t seqs, uint64_t rows) const override {
    size_t n = 4 * (2 * seqs + rows / kLatentTileRows + 1);
    for (const TileSet &s : tile_sets_) n += 4 * (seqs + rows / s.positions + 1);
    return n + 4 * (2 * seqs + rows / kGlaChunk + 1);
  }
  int fill_tiles(const BatchView &b, uint32_t *t, typename Base::Meta &mt) override;
  int fill_latent_tiles(const BatchView &b, uint32_t *t, typename Base::Meta &mt);
  int fill_gla_chunks(const BatchView &b, uint32_t *t, size_t at);
  bool expands(const Layer &L) const { return DTypeOf<T>::is_bf16 && L.latent() && latent_prefill_supported(L.ls); }
  bool tuned(const Layer &L) const { return DTypeOf<T>::is_bf16 && L.latent() && latent_decode_supported(L.ls); }
  uint32_t context_splits(const Layer &L, uint32_t rows) const {
    if (L.attention()) {
      uint32_t s = decode_form_splits(L.kv, L.d.heads, rows, L.form.range.most(meta_.max_position));
      while (s > 1 && decode_scratch_floats(rows, L.d.heads, L.kv.v_dim(), s) > scratch_floats_) --s;
      return s;
    }
    uint32_t s = latent_decode_splits(L.ls, rows, meta_.max_position);
    while (s > 1 && latent_decode_scratch_floats(L.ls, rows, s) > scratch_floats_) --s;
    return s;
  }
  StateBatch state_batch() const {
    const uint32_t *x = d_meta_ + meta_.extra, S = meta_.seqs;
    return StateBatch{x, x + S + 1, x + 2 * S + 1, d_meta_ + meta_.seq_of_row, meta_.rows, S, meta_.decode};
  }
  AttnBatch attn_batch() const {
    const uint32_t *m = d_meta_;
    return AttnBatch{m + meta_.positions, m + meta_.seq_of_row, m + meta_.tables, m + meta_.offsets, meta_.rows, meta_.max_position};
  }
  // The token mixer of one layer: x -> the first mix_out columns of cat_. Names the gate of its output in *y (gated post-norm blocks).
  int mixer(const Layer &L, const T *x, SublayerOutput *y = nullptr);
  int latent_attention(const Layer &L, const GemmPlan &p, size_t slab);
  int attention(const Layer &L, const GemmPlan &p, size_t slab);
  int linear_attention(const Layer &L, const GemmPlan &p, size_t slab);
  // The up half of a dense feed-forward, activated: x -> act (row stride ld).
  int dense_up(const Layer &L, const T *x, T *act, uint32_t ld);
  int mixture(const Layer &L, const T *x, SublayerOutput *y);
  // y's gate: columns from `at` on of a product of `n` columns in partial_.
  void set_gate(const GemmPlan &p, uint32_t n, uint32_t at, const float *bias, SublayerOutput *y) const {
    y->gate = partial_ + at, y->gate_bias = bias, y->gate_splits = p.out_slabs, y->gate_ld = n, y->gate_stride = (size_t)meta_.rows * n;
  }

  OrionLayeredDesc d_;
  std::vector<OrionLayerDesc> specs_;
  OrionModelDesc desc_;
  std::vector<Layer> layers_;         // in the order in which they run
  std::vector<uint32_t> first_run_;   // of every layer of the list
  float *loop_step_ = nullptr;        // [passes][hidden]
  T *pairs_ = nullptr, *places_ = nullptr;  // further tables of the embedding: [buckets + 1][hidden], [learned_positions][hidden]
  uint32_t *history_ = nullptr;             // [blocks][block_size]: token of every cache slot
  std::vector<std::string> got_;
  float *final_norm_ = nullptr;
  T *head_ = nullptr;                        // an output matrix of its own
  T *conv_m_ = nullptr, *conv_f_ = nullptr;  // inputs of the mixer and the feed-forward
  T *cat_ = nullptr;                         // their activations, side by side (sandwich: one after the other)
  float *out_partial_ = nullptr;             // gated post-norm block: products beside those in partial_, which hold the gate
  T *qbuf_ = nullptr;
  T *qa_ = nullptr;           // queries of decoding rows in the latent space
  float *gate_ = nullptr;     // factors of the heads' outputs
  T *value_gate_ = nullptr;   // factors of their values
  float *scratch_ = nullptr;  // partial results of decode attention per context split
  size_t scratch_floats_ = 0;
  MoeBuffers<T> moe_;
  uint32_t few_rows_ = 0;     // rows of this batch that decode
  // Prompt portions of this batch (their descriptions follow the tiles in the batch metadata) and the expanded rows.
  uint32_t portions_ = 0, longest_ = 0, ext_rows_ = 0, ext_cap_ = 0;
  T *ext_latents_ = nullptr, *ext_rot_ = nullptr, *ext_kv_ = nullptr;
  // Prompt portions in tiles for the attention kernels, one list per number of positions in a tile.
  struct TileSet {
    uint32_t positions, count;
    size_t offset;  // words from the start of the tile metadata
  };
  std::vector<TileSet> tile_sets_;
  // The same portions in chunks for linear attention: counts, place of the lists in the tile metadata, scratch.
  uint32_t gla_chunks_ = 0, gla_portions_ = 0;
  size_t gla_at_ = 0, gla_scratch_bytes_ = 0;
  void *gla_scratch_ = nullptr;
  struct Rope {
    double base, factor, original, fast, slow;
    uint32_t dims;
    float *cos, *sin;
  };
  std::vector<Rope> ropes_;
  struct QueryFactors {
    double coef, every;
    float *table;  // [positions]
  };
  std::vector<QueryFactors> query_factors_;
  // What each state slot holds: the number of tokens its state covers and which of its two copies is current.
  struct Slot {
    uint64_t tokens = 0;
    uint32_t copy = 0;
    bool live = false;
  };
  std::vector<Slot> slots_;
};

}  // namespace orion
