// Layer-list models: decoders whose layers are listed one by one, each with its own token mixer and sizes. A
// layer is parallel: one norm, two short causal convolutions of its output, the mixer on one and the
// feed-forward on the other, both results added to the residual stream. What a sequence carries from step to
// step is the paged latent cache of its attention layers and, in a state slot, the recurrences' states
// and the convolutions' last inputs.
//
// Per layer: the mixer and the feed-forward write their activations next to each other into one buffer, and
// their output matrices are stored side by side along k, so the two sublayers end in a single projection
// whose accumulator adds them.
#include "step_model.h"

#include <cmath>
#include <string>

namespace orion {
namespace {

constexpr uint32_t pad8(uint32_t n) { return (n + 7) / 8 * 8; }
// The same, to an odd number of groups of 8 (rows that follow one another in shared memory then start in
// different banks).
constexpr uint32_t odd_groups(uint32_t n) { return pad8(n) / 8 % 2 ? pad8(n) : pad8(n) + 8; }

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
    desc_.max_position_embeddings = d.max_position_embeddings, desc_.rms_norm_eps = (float)d.norm_eps, desc_.tied_lm_head = 1;
    desc_.num_blocks = d.num_blocks, desc_.block_size = d.block_size, desc_.compute_dtype = d.compute_dtype;
    desc_.max_batch_tokens = d.max_batch_tokens, desc_.max_batch_sequences = d.max_batch_sequences, desc_.tp_world = 1;
  }

  ~LayeredModel() override {
    cudaSetDevice(ordinal_);
    if (stream_) cudaStreamSynchronize(stream_);
    for (T *p : {ext_latents_, ext_rot_, ext_kv_})
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
  uint32_t num_state_slots() const override { return d_.num_state_slots; }
  const OrionModelDesc &desc() const override { return desc_; }

 private:
  struct Layer {
    OrionLayerDesc d;
    LatentShape ls{};
    uint32_t mix_in = 0, mix_out = 0, ff_at = 0, cat = 0;  // joint projection columns, mixer output, columns of the joint output projection
    float *norm = nullptr, *mix_bias = nullptr, *latent_norm = nullptr;
    T *conv1 = nullptr, *conv2 = nullptr, *w_mix = nullptr, *w_up = nullptr, *w_out = nullptr, *w_uk = nullptr, *w_uv = nullptr;
    T *conv_state = nullptr;     // [2 * slots][taps - 1][hidden]
    float *rec_state = nullptr;  // [2 * slots][width]
    T *cache = nullptr;          // [blocks][block_size][row_stride]
    const float *rope_cos = nullptr, *rope_sin = nullptr;
    bool attention() const { return d.mixer == ORION_MIXER_LATENT_ATTENTION; }
  };
  // Where a checkpoint tensor goes: rows x cols of it into a matrix of row stride `ld` (dst) or a vector (vec).
  struct Place {
    T *dst = nullptr;
    float *vec = nullptr;
    uint64_t rows = 0, cols = 0, ld = 0;
    uint32_t index = 0;
    bool matrix = true, transposed = false;  // transposed: kept as [cols][rows]
  };
  bool place(const std::string &name, Place *p) const;
  std::vector<std::string> tensor_names() const;

  int run_step_body(bool want_argmax, int part) override;
  bool graph_eligible() const override {
    return g_step_graph && DTypeOf<T>::is_bf16 && meta_.decode && !meta_.zero_count && !prof_on_ && only_mask_ == 0 &&
           residual_norm_conv_supported(d_.hidden_size, d_.conv_taps);
  }
  void graph_plan(uint32_t *splits, uint32_t *blocks_per_split) const override {
    // the context splits of every attention layer, folded into one word
    uint32_t h = 2166136261u;
    for (const Layer &L : layers_)
      if (tuned(L)) h = (h ^ context_splits(L, meta_.rows)) * 16777619u;
    *splits = h, *blocks_per_split = 0;
  }
  int check_batch(const BatchView &b) override;
  // [first row of each sequence, S + 1][state copy to read, S][to write, S][rows that decode, kFewRows * S]
  size_t extra_words(uint64_t seqs) const override { return (3 + kFewRows) * seqs + 1; }
  void fill_extra(const BatchView &b, uint32_t *w) override;
  void step_done(const BatchView &b) override;
  int poll_errors() override {
    ORION_TRY(Base::poll_errors());
    uint32_t code = 0;
    if (DTypeOf<T>::is_bf16) ORION_TRY(latent_poll_error(&code));
    if (DTypeOf<T>::is_bf16 && !code) ORION_TRY(latent_prefill_poll_error(&code));
    if (code) return set_error(ORION_ERR_BACKEND, "backend cuda failed at latent attention: a bounded pipeline wait ran out (code %u)", code);
    return ORION_OK;
  }
  // Sequences with at most this many rows in a batch decode: each row reads the cache by itself.
  static constexpr uint32_t kFewRows = 8;
  size_t tile_words(uint64_t seqs, uint64_t rows) const override { return 4 * (2 * seqs + rows / kLatentTileRows + 1); }
  int fill_tiles(const BatchView &b, uint32_t *t, typename Base::Meta &mt) override;
  bool expands(const Layer &L) const { return DTypeOf<T>::is_bf16 && L.attention() && latent_prefill_supported(L.ls); }
  bool tuned(const Layer &L) const { return DTypeOf<T>::is_bf16 && L.attention() && latent_decode_supported(L.ls); }
  uint32_t context_splits(const Layer &L, uint32_t rows) const {
    uint32_t s = latent_decode_splits(L.ls, rows, meta_.max_position);
    while (s > 1 && latent_decode_scratch_floats(L.ls, rows, s) > scratch_floats_) --s;
    return s;
  }
  StateBatch state_batch() const {
    const uint32_t *x = d_meta_ + meta_.extra, S = meta_.seqs;
    return StateBatch{x, x + S + 1, x + 2 * S + 1, d_meta_ + meta_.seq_of_row, meta_.rows, S, meta_.decode};
  }
  int mixer(const Layer &L, const StateBatch &sb, const AttnBatch &ab);

  OrionLayeredDesc d_;
  std::vector<OrionLayerDesc> specs_;
  OrionModelDesc desc_;
  std::vector<Layer> layers_;
  std::vector<std::string> got_;
  float *final_norm_ = nullptr;
  T *conv_m_ = nullptr, *conv_f_ = nullptr;  // inputs of the mixer and the feed-forward
  T *cat_ = nullptr;                         // their activations, side by side
  T *qbuf_ = nullptr;
  T *qa_ = nullptr;           // queries of decoding rows in the latent space
  float *scratch_ = nullptr;  // their weighted latents per context split
  size_t scratch_floats_ = 0;
  uint32_t few_rows_ = 0;     // rows of this batch that decode
  // Prompt portions of this batch (their descriptions follow the tiles in the batch metadata) and the expanded rows.
  uint32_t portions_ = 0, longest_ = 0, ext_rows_ = 0, ext_cap_ = 0;
  T *ext_latents_ = nullptr, *ext_rot_ = nullptr, *ext_kv_ = nullptr;
  struct Rope {
    double base;
    uint32_t dims;
    float *cos, *sin;
  };
  std::vector<Rope> ropes_;
  // What each state slot holds: the number of tokens its state covers and which of its two copies is current.
  struct Slot {
    uint64_t tokens = 0;
    uint32_t copy = 0;
    bool live = false;
  };
  std::vector<Slot> slots_;
};

template <typename T>
int LayeredModel<T>::init() {
  const OrionLayeredDesc &d = d_;
  if (d.hidden_size == 0 || d.vocab_size == 0 || d.num_layers == 0 || d.conv_taps == 0)
    return set_error(ORION_ERR_MODEL, "config.json is malformed: a model dimension is zero");
  if (d.block_size == 0 || d.max_batch_tokens == 0 || d.max_batch_sequences == 0 || d.num_state_slots == 0)
    return set_error(ORION_ERR_INVALID_REQUEST,
                     "block_size, max_batch_tokens, max_batch_sequences and num_state_slots must be non-zero");
  for (uint32_t i = 0; i < d.num_layers; ++i) {
    const OrionLayerDesc &s = specs_[i];
    if (s.mixer == ORION_MIXER_MIN_GRU ? s.width == 0
                                       : s.mixer != ORION_MIXER_LATENT_ATTENTION || s.heads == 0 || s.dim + s.rot_dim == 0 ||
                                             s.value_dim == 0 || s.kv_rank == 0)
      return set_error(ORION_ERR_MODEL, "config.json is malformed: layer %u has an unknown mixer or a size of zero", i);
    if (s.mixer == ORION_MIXER_LATENT_ATTENTION && (s.rope_dims % 2 != 0 || s.rope_dims > s.rot_dim))
      return set_error(ORION_ERR_MODEL, "config.json is malformed: layer %u rotates %u of %u dimensions", i, s.rope_dims, s.rot_dim);
  }
  ORION_TRY(Base::init_step({d.hidden_size, d.vocab_size, d.max_position_embeddings, d.num_blocks, d.block_size, d.max_batch_tokens,
                             d.max_batch_sequences}));
  const size_t H = d.hidden_size, copies = 2 * (size_t)d.num_state_slots, keep = d.conv_taps - 1, rows = d.max_batch_tokens;
  auto zeroed = [&](auto **p, size_t n) -> int {
    ORION_TRY(alloc(p, n));
    ORION_CUDA_CHECK("clear buffer", cudaMemsetAsync(*p, 0, (n ? n : 1) * sizeof(**p), stream_));
    return ORION_OK;
  };
  size_t cat = 0, qcols = 0;
  layers_.resize(d.num_layers);
  for (uint32_t i = 0; i < d.num_layers; ++i) {
    Layer &L = layers_[i];
    L.d = specs_[i];
    const OrionLayerDesc &s = L.d;
    ORION_TRY(alloc(&L.norm, H));
    ORION_TRY(alloc(&L.conv1, H * d.conv_taps));
    ORION_TRY(zeroed(&L.conv_state, copies * keep * H));
    if (L.attention()) {
      L.ls = LatentShape{s.heads, s.dim, s.rot_dim, s.value_dim, s.kv_rank, s.window, s.rope_dims, d.block_size,
                         odd_groups(s.kv_rank + s.rot_dim), (float)s.scale, (float)d.norm_eps};
      L.mix_in = L.ls.cols(), L.mix_out = L.ls.out_cols();
      ORION_TRY(alloc(&L.latent_norm, s.kv_rank));
      ORION_TRY(alloc(&L.w_uk, (size_t)s.heads * (s.dim + s.value_dim) * s.kv_rank));  // one matrix for the expansion of prompts
      L.w_uv = L.w_uk + (size_t)s.heads * s.dim * s.kv_rank;
      ORION_TRY(zeroed(&L.cache, (size_t)d.num_blocks * d.block_size * L.ls.row_stride));
      qcols = std::max(qcols, (size_t)L.ls.q_cols());
      const Rope *r = nullptr;
      for (const Rope &x : ropes_)
        if (x.base == s.rope_base && x.dims == s.rope_dims) r = &x;
      if (!r) {
        const size_t half = s.rope_dims / 2, n = (size_t)d.max_position_embeddings * half;
        std::vector<float> c(n ? n : 1), sn(n ? n : 1);
        for (size_t p = 0; p < d.max_position_embeddings; ++p)
          for (size_t k = 0; k < half; ++k) {
            const double angle = (double)p * std::pow(s.rope_base, -2.0 * (double)k / (double)s.rope_dims);
            c[p * half + k] = (float)std::cos(angle);
            sn[p * half + k] = (float)std::sin(angle);
          }
        Rope fresh{s.rope_base, s.rope_dims, nullptr, nullptr};
        ORION_TRY(alloc(&fresh.cos, n));
        ORION_TRY(alloc(&fresh.sin, n));
        ORION_CUDA_CHECK("upload rope", cudaMemcpy(fresh.cos, c.data(), n * sizeof(float), cudaMemcpyHostToDevice));
        ORION_CUDA_CHECK("upload rope", cudaMemcpy(fresh.sin, sn.data(), n * sizeof(float), cudaMemcpyHostToDevice));
        ropes_.push_back(fresh);
        r = &ropes_.back();
      }
      L.rope_cos = r->cos, L.rope_sin = r->sin;
    } else {
      L.mix_in = 3 * s.width, L.mix_out = s.width;
      ORION_TRY(alloc(&L.mix_bias, 2 * (size_t)s.width));
      ORION_TRY(zeroed(&L.rec_state, copies * s.width));
    }
    ORION_TRY(alloc(&L.w_mix, (size_t)L.mix_in * H));
    // both parts of the joint output projection start at a multiple of 8 columns; the weights of the columns
    // between them are zero
    L.ff_at = pad8(L.mix_out);
    L.cat = L.ff_at + pad8(s.ffn_dim);
    ORION_TRY(zeroed(&L.w_out, H * L.cat));
    if (s.ffn_dim) {
      ORION_TRY(alloc(&L.conv2, H * d.conv_taps));
      ORION_TRY(alloc(&L.w_up, (size_t)s.ffn_dim * H));
    }
    cat = std::max(cat, (size_t)L.cat);
    constexpr bool kBf16 = DTypeOf<T>::is_bf16;
    for (const auto &nk : {std::make_pair(L.mix_in, (uint32_t)H), std::make_pair(s.ffn_dim, (uint32_t)H), std::make_pair((uint32_t)H, L.cat)})
      if (nk.first) partial_floats_ = std::max(partial_floats_, gemm_partial_floats(kBf16, (uint32_t)rows, nk.first, nk.second));
  }
  ORION_TRY(alloc(&embed_, (size_t)d.vocab_size * H));
  ORION_TRY(alloc(&final_norm_, H));
  ORION_TRY(alloc(&partial_, partial_floats_));
  ORION_TRY(alloc(&conv_m_, rows * H));
  ORION_TRY(alloc(&conv_f_, rows * H));
  ORION_TRY(zeroed(&cat_, rows * cat));  // columns that nobody writes meet zero weights and must be finite
  ORION_TRY(alloc(&qbuf_, rows * qcols));
  size_t qa = 0;
  const uint32_t few = (uint32_t)std::min<uint64_t>(rows, (uint64_t)kFewRows * d.max_batch_sequences);
  for (const Layer &L : layers_) {
    if (!tuned(L)) continue;
    qa = std::max(qa, (size_t)few * L.ls.heads * L.ls.kv_cols());
    for (uint32_t r = 1; r <= few; ++r)
      scratch_floats_ = std::max(scratch_floats_, latent_decode_scratch_floats(L.ls, r, latent_decode_splits(L.ls, r, d.max_position_embeddings)));
  }
  ORION_TRY(alloc(&qa_, qa));
  ORION_TRY(alloc(&scratch_, scratch_floats_));
  slots_.resize(d.num_state_slots);
  ORION_CUDA_CHECK("model init", cudaStreamSynchronize(stream_));
  return ORION_OK;
}

template <typename T>
bool LayeredModel<T>::place(const std::string &name, Place *p) const {
  const uint64_t H = d_.hidden_size;
  auto matrix = [&](T *dst, uint64_t rows, uint64_t cols, uint64_t ld = 0) {
    p->dst = dst, p->rows = rows, p->cols = cols, p->ld = ld ? ld : cols, p->matrix = true;
    return rows > 0;
  };
  auto filters = [&](T *dst) {
    p->transposed = true;
    return matrix(dst, H, d_.conv_taps);
  };
  auto vector = [&](float *dst, uint64_t n) {
    p->vec = dst, p->rows = 1, p->cols = n, p->matrix = false;
    return n > 0;
  };
  if (name == "embed") return matrix(embed_, d_.vocab_size, H);
  if (name == "final.norm") return vector(final_norm_, H);
  unsigned i = 0;
  int used = 0;
  if (sscanf(name.c_str(), "l%u.%n", &i, &used) != 1 || used == 0 || i >= layers_.size()) return false;
  const std::string rest = name.substr((size_t)used);
  const Layer &L = layers_[i];
  const OrionLayerDesc &s = L.d;
  p->index = i;
  if (rest == "norm1") return vector(L.norm, H);
  if (rest == "canon1") return filters(L.conv1);
  if (s.ffn_dim) {
    if (rest == "canon2") return filters(L.conv2);
    if (rest == "mlp.up") return matrix(L.w_up, s.ffn_dim, H);
    if (rest == "mlp.down") return matrix(L.w_out + L.ff_at, H, s.ffn_dim, L.cat);
  }
  if (rest == "mix.o") return matrix(L.w_out, H, L.mix_out, L.cat);
  if (L.attention()) {
    const LatentShape &a = L.ls;
    if (rest == "mix.q") return matrix(L.w_mix, a.q_cols(), H);
    if (rest == "mix.dkv") return matrix(L.w_mix + a.q_cols() * H, a.kv_cols(), H);
    if (rest == "mix.g") return matrix(L.w_mix + (a.q_cols() + a.kv_cols()) * H, a.out_cols(), H);
    if (rest == "mix.dkv.norm") return vector(L.latent_norm, s.kv_rank);
    if (rest == "mix.uk") return matrix(L.w_uk, (uint64_t)s.heads * s.dim, s.kv_rank);
    if (rest == "mix.uv") return matrix(L.w_uv, (uint64_t)s.heads * s.value_dim, s.kv_rank);
    return false;
  }
  if (rest == "mix.z") return matrix(L.w_mix, s.width, H);
  if (rest == "mix.x") return matrix(L.w_mix + s.width * H, s.width, H);
  if (rest == "mix.g") return matrix(L.w_mix + 2 * (uint64_t)s.width * H, s.width, H);
  if (rest == "mix.z.b") return vector(L.mix_bias, s.width);
  if (rest == "mix.x.b") return vector(L.mix_bias + s.width, s.width);
  return false;
}

template <typename T>
std::vector<std::string> LayeredModel<T>::tensor_names() const {
  std::vector<std::string> names = {"embed", "final.norm"};
  for (uint32_t i = 0; i < d_.num_layers; ++i)
    for (const char *rest : {"norm1", "canon1", "canon2", "mlp.up", "mlp.down", "mix.o", "mix.q", "mix.dkv", "mix.dkv.norm", "mix.uk",
                             "mix.uv", "mix.g", "mix.z", "mix.x", "mix.z.b", "mix.x.b"}) {
      const std::string name = "l" + std::to_string(i) + "." + rest;
      if (uses_tensor(name.c_str())) names.push_back(name);
    }
  return names;
}

template <typename T>
int LayeredModel<T>::load_tensor(const char *name, int dtype, const uint64_t *shape, int ndim, const void *data) {
  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  if (dtype_size(dtype) == 0) return set_error(ORION_ERR_MODEL, "unsupported dtype %d (tensor `%s`)", dtype, name);
  if (!data || ndim < 1 || ndim > 2) return set_error(ORION_ERR_MODEL, "tensor `%s` has rank %d", name, ndim);
  Place p;
  if (!place(name, &p)) return set_error(ORION_ERR_MODEL, "tensor `%s` is not part of the model", name);
  const uint64_t R = ndim == 2 ? shape[0] : 1, C = ndim == 2 ? shape[1] : shape[0];
  if (R != p.rows || C != p.cols || (ndim == 2) != p.matrix)
    return set_error(ORION_ERR_MODEL, "tensor `%s` has shape [%llu, %llu], expected [%llu, %llu]", name, (unsigned long long)R,
                     (unsigned long long)C, (unsigned long long)p.rows, (unsigned long long)p.cols);
  finalized_ = false;
  if (!p.matrix) {
    ORION_TRY(upload_slice(nullptr, p.vec, data, dtype, C, 0, 1, 0, C));
  } else if (p.ld == C && !p.transposed) {
    ORION_TRY(upload_slice(p.dst, nullptr, data, dtype, C, 0, R, 0, C));
  } else {  // a column block of a wider matrix, or filters
    T *tmp = nullptr;
    ORION_CUDA_CHECK("allocate staging", cudaMalloc(&tmp, R * C * sizeof(T)));
    int rc = upload_slice(tmp, nullptr, data, dtype, C, 0, R, 0, C);
    if (rc == ORION_OK)
      rc = p.transposed ? launch_transpose<T>(tmp, p.dst, (uint32_t)R, (uint32_t)C, stream_)
                        : launch_copy_rows_strided<T>(tmp, p.dst, R, C, p.ld, stream_);
    const cudaError_t e = cudaStreamSynchronize(stream_);
    cudaFree(tmp);
    ORION_TRY(rc);
    ORION_CUDA_CHECK("upload tensor", e);
  }
  if (std::find(got_.begin(), got_.end(), name) == got_.end()) got_.push_back(name);
  return ORION_OK;
}

template <typename T>
int LayeredModel<T>::finalize() {
  for (const std::string &n : tensor_names())
    if (std::find(got_.begin(), got_.end(), n) == got_.end()) return set_error(ORION_ERR_MODEL, "missing tensor `%s`", n.c_str());
  lm_head_ = embed_;
  finalized_ = true;
  return ORION_OK;
}

template <typename T>
int LayeredModel<T>::init_random(uint64_t seed, float std) {
  // N(0, std) matrices, norm gains 1, zero biases; the filters keep most of the current row's weight out of
  // the sum like a trained one would (std 0.1 per tap).
  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  for (const std::string &n : tensor_names()) {
    Place p;
    place(n, &p);
    if (!p.matrix) {
      ORION_TRY(set_constant(p.vec, p.cols, n.size() > 2 && n.compare(n.size() - 2, 2, ".b") == 0 ? 0.0f : 1.0f));
    } else if (p.ld == p.cols) {
      ORION_TRY(fill_random(p.dst, p.rows * p.cols, seed, n.find(".canon") != std::string::npos ? 0.1f : std));
    } else {
      T *tmp = nullptr;
      ORION_CUDA_CHECK("allocate staging", cudaMalloc(&tmp, p.rows * p.cols * sizeof(T)));
      int rc = fill_random(tmp, p.rows * p.cols, seed, std);
      if (rc == ORION_OK) rc = launch_copy_rows_strided<T>(tmp, p.dst, p.rows, p.cols, p.ld, stream_);
      const cudaError_t e = cudaStreamSynchronize(stream_);
      cudaFree(tmp);
      ORION_TRY(rc);
      ORION_CUDA_CHECK("init_random", e);
    }
    got_.push_back(n);
  }
  ORION_CUDA_CHECK("init_random", cudaStreamSynchronize(stream_));
  return finalize();
}

template <typename T>
int LayeredModel<T>::check_batch(const BatchView &b) {
  const uint64_t S = b.num_sequences;
  if (!b.state_slots || b.num_state_slots != S)
    return set_error(ORION_ERR_INVALID_REQUEST, "this model needs a state slot for each of the %llu sequences", (unsigned long long)S);
  std::vector<bool> taken(slots_.size(), false);
  uint64_t row = 0;
  for (uint64_t s = 0; s < S; ++s) {
    const uint32_t slot = b.state_slots[s];
    const uint64_t n = b.slot_token_counts[s];
    if (n == 0) return set_error(ORION_ERR_INTERNAL, "a scheduled sequence contributed zero tokens");
    if (slot >= slots_.size())
      return set_error(ORION_ERR_INTERNAL, "state slot %u out of range (have %zu)", slot, slots_.size());
    if (taken[slot]) return set_error(ORION_ERR_INTERNAL, "state slot %u is named twice in one batch", slot);
    taken[slot] = true;
    for (uint64_t i = 1; i < n; ++i)
      if (b.positions[row + i] != b.positions[row] + i)
        return set_error(ORION_ERR_INTERNAL, "the positions of sequence %llu are not consecutive", (unsigned long long)s);
    if (b.positions[row] != 0 && (!slots_[slot].live || slots_[slot].tokens != b.positions[row]))
      return set_error(ORION_ERR_INTERNAL, "sequence %llu goes on at position %u but its state covers %llu tokens",
                       (unsigned long long)s, b.positions[row], (unsigned long long)(slots_[slot].live ? slots_[slot].tokens : 0));
    row += n;
  }
  return ORION_OK;
}

template <typename T>
void LayeredModel<T>::fill_extra(const BatchView &b, uint32_t *w) {
  const uint64_t S = b.num_sequences;
  uint32_t *first = w, *read = w + S + 1, *write = read + S, *few = write + S;
  uint64_t row = 0;
  few_rows_ = portions_ = 0;
  for (uint64_t s = 0; s < S; ++s) {
    const uint32_t slot = b.state_slots[s], copy = slots_[slot].copy;
    first[s] = (uint32_t)row;
    read[s] = b.positions[row] == 0 ? kNoState : 2 * slot + copy;
    write[s] = 2 * slot + (copy ^ 1u);
    if (b.slot_token_counts[s] <= kFewRows)
      for (uint64_t i = 0; i < b.slot_token_counts[s]; ++i) few[few_rows_++] = (uint32_t)(row + i);
    row += b.slot_token_counts[s];
  }
  first[S] = (uint32_t)row;
}

// Portions and tiles of the sequences that bring more than a few rows, and room for their expanded rows.
template <typename T>
int LayeredModel<T>::fill_tiles(const BatchView &b, uint32_t *t, typename Base::Meta &mt) {
  uint64_t reach = 0, wide = 0, rank = 0, rot = 0;  // tokens before a portion that some window reaches; buffer widths
  bool any = false;
  for (const Layer &L : layers_) {
    if (!expands(L)) continue;
    any = true;
    reach = std::max(reach, L.d.window ? (uint64_t)L.d.window - 1 : UINT64_MAX);
    wide = std::max(wide, (uint64_t)L.d.heads * (L.d.dim + L.d.value_dim));
    rank = std::max(rank, (uint64_t)L.d.kv_rank);
    rot = std::max(rot, (uint64_t)L.d.rot_dim);
  }
  if (!any) return ORION_OK;
  auto *portions = reinterpret_cast<LatentPortion *>(t);
  auto *tiles = reinterpret_cast<LatentTile *>(t + 4 * b.num_sequences);
  uint64_t row = 0, ext = 0;
  longest_ = 0;
  for (uint64_t s = 0; s < b.num_sequences; ++s) {
    const uint64_t n = b.slot_token_counts[s];
    if (n > kFewRows) {
      const uint64_t start = b.positions[row], before = std::min(start, reach);
      if (ext + before + n > INT32_MAX) return set_error(ORION_ERR_INVALID_REQUEST, "prompt portions reach too many tokens");
      portions[portions_++] = LatentPortion{(uint32_t)s, (uint32_t)ext, (uint32_t)(start - before), (uint32_t)(before + n)};
      longest_ = std::max(longest_, (uint32_t)(before + n));
      for (uint64_t i = 0; i < n; i += kLatentTileRows)
        tiles[mt.num_tiles++] = LatentTile{(uint32_t)(row + i), (uint32_t)std::min<uint64_t>(kLatentTileRows, n - i), (uint32_t)(start + i),
                                           (int32_t)((int64_t)(ext + before) - (int64_t)start)};
      ext += before + n;
    }
    row += n;
  }
  ext_rows_ = (uint32_t)ext;
  if (ext > ext_cap_) {
    uint64_t cap = 1024;
    while (cap < ext) cap *= 2;
    ext_cap_ = 0;
    for (auto [buf, width] : {std::make_pair(&ext_latents_, rank), std::make_pair(&ext_rot_, rot), std::make_pair(&ext_kv_, wide)}) {
      if (*buf) cudaFree(*buf);  // the previous step has ended
      *buf = nullptr;
      const size_t bytes = std::max<size_t>(1, cap * width) * sizeof(T);
      ORION_CUDA_CHECK("allocate expanded rows", cudaMalloc(buf, bytes));
      ORION_CUDA_CHECK("allocate expanded rows", cudaMemsetAsync(*buf, 0, bytes, stream_));  // masked keys must be finite
    }
    ext_cap_ = (uint32_t)cap;
  }
  return ORION_OK;
}

template <typename T>
void LayeredModel<T>::step_done(const BatchView &b) {
  uint64_t row = 0;
  for (uint64_t s = 0; s < b.num_sequences; ++s) {
    Slot &x = slots_[b.state_slots[s]];
    x.tokens = (uint64_t)b.positions[row] + b.slot_token_counts[s];
    x.copy ^= 1u;
    x.live = true;
    row += b.slot_token_counts[s];
  }
}

// The token mixer of one layer: conv_m_ -> the first mix_out columns of cat_.
template <typename T>
int LayeredModel<T>::mixer(const Layer &L, const StateBatch &sb, const AttnBatch &ab) {
  const uint32_t Tn = meta_.rows, H = d_.hidden_size;
  const GemmPlan p = plan_for(Tn, L.mix_in, H, H);
  const size_t slab = (size_t)Tn * L.mix_in;
  ORION_TRY(timed(kProfGemm, [&] { return launch_gemm<T>(conv_m_, H, L.w_mix, H, partial_, Tn, L.mix_in, H, p, stream_); }));
  if (!L.attention())
    return timed(kProfAttention, [&] { return launch_min_gru<T>(partial_, p.out_slabs, slab, L.mix_bias, L.rec_state, sb, cat_, L.cat, L.d.width, stream_); });
  ORION_TRY(timed(kProfAttention, [&] {
    return launch_latent_prepare<T>(partial_, p.out_slabs, slab, L.latent_norm, L.rope_cos, L.rope_sin, ab.query_positions,
                                    d_meta_ + meta_.slot_block, d_meta_ + meta_.slot_slot, qbuf_, L.cache, L.ls, Tn, stream_);
  }));
  if constexpr (DTypeOf<T>::is_bf16) {
    if ((few_rows_ == 0 || tuned(L)) && (few_rows_ == Tn || expands(L))) {
      const uint32_t *first = d_meta_ + meta_.extra, *few = first + 3 * meta_.seqs + 1;
      if (few_rows_ > 0) {
        const uint32_t sp = context_splits(L, few_rows_);
        ORION_TRY(timed(kProfAttention, [&] { return launch_latent_absorb(qbuf_, L.w_uk, few, few_rows_, qa_, L.ls, stream_); }));
        ORION_TRY(timed(kProfAttention, [&] {
          return launch_latent_decode(qa_, L.cache, L.w_uv, partial_, p.out_slabs, slab, few, first, few_rows_, ab, sp, scratch_, L.ls, cat_,
                                      L.cat, stream_);
        }));
      }
      if (portions_ > 0) {
        const auto *portions = reinterpret_cast<const LatentPortion *>(d_meta_ + meta_.tiles);
        const auto *tiles = reinterpret_cast<const LatentTile *>(d_meta_ + meta_.tiles + 4 * meta_.seqs);
        const uint32_t wide = L.d.heads * (L.d.dim + L.d.value_dim);
        ORION_TRY(timed(kProfAttention, [&] {
          return launch_latent_gather(L.cache, ab.tables_flat, ab.table_offsets, portions, portions_, longest_, ext_latents_, ext_rot_, L.ls, stream_);
        }));
        ORION_TRY(timed(kProfGemm, [&] {
          return launch_gemm_act(ext_latents_, L.d.kv_rank, L.w_uk, L.d.kv_rank, ext_kv_, wide, ext_rows_, wide, L.d.kv_rank, kGemmStore, stream_);
        }));
        ORION_TRY(timed(kProfAttention, [&] {
          return launch_latent_prefill(qbuf_, ext_kv_, ext_rot_, ext_cap_, partial_, p.out_slabs, slab, tiles, meta_.num_tiles, L.ls, cat_, L.cat,
                                       stream_);
        }));
      }
      return ORION_OK;
    }
  }
  return timed(kProfAttention, [&] {
    return launch_latent_attention_generic<T>(qbuf_, L.cache, L.w_uk, L.w_uv, partial_, p.out_slabs, slab, L.ls, ab, cat_, L.cat, stream_);
  });
}

template <typename T>
int LayeredModel<T>::run_step_body(bool want_argmax, int part) {
  const uint32_t Tn = meta_.rows, H = d_.hidden_size, taps = d_.conv_taps;
  const uint32_t *m = d_meta_, *tokens = m + meta_.tokens;
  const float eps = (float)d_.norm_eps;
  const StateBatch sb = state_batch();
  const AttnBatch ab{m + meta_.positions, m + meta_.seq_of_row, m + meta_.tables, m + meta_.offsets, Tn, meta_.max_position};
  // Decode batches take the residual add (or the embedding), the norm and the convolutions in one kernel.
  const bool fused = sb.single && residual_norm_conv_supported(H, taps);
  GemmPlan out{};
  for (uint32_t l = 0; part != 2 && l < d_.num_layers; ++l) {
    const Layer &L = layers_[l];
    T *ff_in = L.d.ffn_dim ? conv_f_ : nullptr;
    if (fused) {
      ORION_TRY(timed(kProfElementwise, [&] {
        return launch_residual_norm_conv<T>(partial_, out.out_slabs, (size_t)Tn * H, l ? nullptr : embed_, tokens, hidden_, L.norm, eps,
                                            L.conv1, L.conv2, taps, L.conv_state, sb, conv_m_, ff_in, H, stream_);
      }));
    } else {
      ORION_TRY(timed(kProfElementwise, [&] {
        return l ? launch_residual_rmsnorm<T>(partial_, out.out_slabs, (size_t)Tn * H, hidden_, L.norm, eps, normed_, nullptr, Tn, H, stream_)
                 : launch_embed_rmsnorm<T>(embed_, tokens, L.norm, eps, hidden_, normed_, Tn, H, stream_);
      }));
      ORION_TRY(timed(kProfElementwise, [&] {
        return launch_causal_conv<T>(normed_, L.conv1, L.conv2, taps, L.conv_state, sb, conv_m_, ff_in, H, stream_);
      }));
    }
    if (L.d.ffn_dim) {
      const uint32_t F = L.d.ffn_dim;
      const GemmPlan p = plan_for(Tn, F, H, H);
      bool in_epilogue = false;
      if constexpr (DTypeOf<T>::is_bf16) {
        if (p.tensor_core && p.splits == 1) {  // GELU in the GEMM epilogue: no partials, no extra launch
          in_epilogue = true;
          ORION_TRY(timed(kProfGemm, [&] { return launch_gemm_act(conv_f_, H, L.w_up, H, cat_ + L.ff_at, L.cat, Tn, F, H, kGemmGelu, stream_); }));
        }
      }
      if (!in_epilogue) {
        ORION_TRY(timed(kProfGemm, [&] { return launch_gemm<T>(conv_f_, H, L.w_up, H, partial_, Tn, F, H, p, stream_); }));
        ORION_TRY(timed(kProfElementwise, [&] {
          return launch_ffn_act<T>(partial_, p.out_slabs, (size_t)Tn * F, nullptr, kActGelu, cat_ + L.ff_at, L.cat, Tn, F, stream_);
        }));
      }
    }
    ORION_TRY(mixer(L, sb, ab));
    out = plan_for(Tn, H, L.cat, L.cat);
    ORION_TRY(timed(kProfGemm, [&] { return launch_gemm<T>(cat_, L.cat, L.w_out, L.cat, partial_, Tn, H, L.cat, out, stream_); }));
  }
  if (part != 2 && meta_.outs > 0)
    ORION_TRY(timed(kProfElementwise, [&] {
      return launch_residual_rmsnorm<T>(partial_, out.out_slabs, (size_t)Tn * H, hidden_, final_norm_, eps, tail_, m + meta_.last_rows,
                                        meta_.outs, H, stream_);
    }));
  if (part == 1 || meta_.outs == 0) return ORION_OK;
  return run_head(want_argmax);
}

template <typename T>
int LayeredModel<T>::fill_kv_random(uint64_t seed, float std) {
  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  for (const Layer &L : layers_)
    if (L.attention()) ORION_TRY(fill_random(L.cache, (size_t)d_.num_blocks * d_.block_size * L.ls.row_stride, seed, std));
  ORION_CUDA_CHECK("fill_kv_random", cudaStreamSynchronize(stream_));
  return ORION_OK;
}

// The latent caches of the attention layers, one after the other: [block][slot][kv_rank + rot_dim].
template <typename T>
int LayeredModel<T>::read_kv(float *out, uint64_t capacity) {
  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  const size_t tokens = (size_t)d_.num_blocks * d_.block_size;
  for (const Layer &L : layers_) {
    if (!L.attention()) continue;
    const size_t cols = L.ls.kv_cols(), stride = L.ls.row_stride, n = tokens * stride;
    if (capacity < tokens * cols) return set_error(ORION_ERR_INVALID_REQUEST, "KV read-back buffer is too small");
    ORION_TRY(ensure_stage(&stage_f32_, &stage_f32_cap_, n * sizeof(float)));
    float *tmp = static_cast<float *>(stage_f32_);
    ORION_TRY(launch_convert_to_f32<T>(L.cache, tmp, n, stream_));
    ORION_CUDA_CHECK("read_kv", cudaMemcpy2DAsync(out, cols * sizeof(float), tmp, stride * sizeof(float), cols * sizeof(float), tokens,
                                                  cudaMemcpyDeviceToHost, stream_));
    ORION_CUDA_CHECK("read_kv", cudaStreamSynchronize(stream_));
    out += tokens * cols;
    capacity -= tokens * cols;
  }
  return ORION_OK;
}

}  // namespace

int create_layered_model(OrionBackend *backend, const OrionLayeredDesc *desc, ModelBase **out) {
  *out = nullptr;
  if (desc->num_layers > 0 && !desc->layers) return set_error(ORION_ERR_INVALID_REQUEST, "null layer list");
  auto make = [&](auto *m) -> int {
    const int rc = m->init();
    if (rc != ORION_OK) { delete m; return rc; }
    *out = m;
    return ORION_OK;
  };
  if (desc->compute_dtype == ORION_DTYPE_F32) return make(new LayeredModel<float>(backend, *desc));
  if (desc->compute_dtype == ORION_DTYPE_BF16) return make(new LayeredModel<bf16>(backend, *desc));
  return set_error(ORION_ERR_MODEL, "unsupported compute dtype %u (f32 and bf16 are implemented)", desc->compute_dtype);
}

}  // namespace orion
