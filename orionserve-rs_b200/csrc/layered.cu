// Layer-list models: sizes, weights, state slots and batch description (layered_step.cu has the kernel sequence).
#include "layered.h"

#include <cmath>

namespace orion {
namespace {

constexpr uint32_t pad8(uint32_t n) { return (n + 7) / 8 * 8; }
// The same, to an odd number of groups of 8 (rows that follow one another in shared memory then start in
// different banks).
constexpr uint32_t odd_groups(uint32_t n) { return pad8(n) / 8 % 2 ? pad8(n) : pad8(n) + 8; }

}  // namespace

template <typename T>
int LayeredModel<T>::check_layer(uint32_t i) const {
  const OrionLayerDesc &s = specs_[i];
  bool sizes = false;
  switch (s.mixer) {
    case ORION_MIXER_MIN_GRU: sizes = s.width > 0; break;
    case ORION_MIXER_LATENT_ATTENTION: sizes = s.heads > 0 && s.dim + s.rot_dim > 0 && s.value_dim > 0 && s.kv_rank > 0; break;
    case ORION_MIXER_GLA: sizes = s.heads > 0 && s.dim > 0 && s.value_dim > 0 && s.decay_rank > 0 && s.decay_tau > 0; break;
    case ORION_MIXER_ATTENTION: sizes = s.heads > 0 && s.kv_heads > 0 && s.heads % s.kv_heads == 0 && s.dim > 0 && s.value_dim > 0; break;
  }
  if (!sizes)
    return set_error(ORION_ERR_MODEL, "config.json is malformed: layer %u has an unknown mixer, a size of zero or uneven groups of heads", i);
  const uint32_t rotates = s.mixer == ORION_MIXER_ATTENTION ? s.dim : s.rot_dim;
  if ((s.mixer == ORION_MIXER_ATTENTION || s.mixer == ORION_MIXER_LATENT_ATTENTION) && (s.rope_dims % 2 != 0 || s.rope_dims > rotates))
    return set_error(ORION_ERR_MODEL, "config.json is malformed: layer %u rotates %u of %u dimensions", i, s.rope_dims, rotates);
  if (s.keys_as_values && (s.mixer != ORION_MIXER_ATTENTION || s.qk_norm != ORION_QK_NORM_ALL_HEADS || s.rope_dims || s.head_gate || s.value_dim != s.dim))
    return set_error(ORION_ERR_MODEL, "layer %u: keys as values come with norms over all heads, without rotation and gates, and values of the keys' size", i);
  if ((s.distance_bias || s.q_temp_every != 0) && !s.keys_as_values)
    return set_error(ORION_ERR_MODEL, "layer %u: distance terms and query factors come with keys as values", i);
  if (s.sinks > ORION_SINK_ZERO || s.q_temp_every < 0) return set_error(ORION_ERR_MODEL, "config.json is malformed: layer %u has an unknown sink or query factor", i);
  const uint64_t outputs = (uint64_t)s.experts + s.router_identity;
  if (s.router_groups && (s.router != ORION_ROUTER_SOFTMAX_RENORM || outputs % s.router_groups || s.router_keep == 0 || s.router_keep > s.router_groups ||
                          s.experts_per_token > outputs / s.router_groups * s.router_keep))
    return set_error(ORION_ERR_MODEL, "config.json is malformed: layer %u uses %u of %llu experts, of %u of %u groups", i, s.experts_per_token,
                     (unsigned long long)outputs, s.router_keep, s.router_groups);
  if (s.experts > 0 && (s.ffn_dim == 0 || s.experts_per_token == 0 || s.experts_per_token > outputs || outputs > kMoeMaxExperts))
    return set_error(ORION_ERR_MODEL, "config.json is malformed: layer %u uses %u of %llu experts of width %u (at most %u experts)", i,
                     s.experts_per_token, (unsigned long long)outputs, s.ffn_dim, kMoeMaxExperts);
  if (s.activation > ORION_ACT_GEGLU_TANH || s.router > ORION_ROUTER_SOFTMAX_RENORM || s.expert_form > ORION_EXPERT_GELU || s.qk_norm > ORION_QK_NORM_PER_HEAD)
    return set_error(ORION_ERR_MODEL, "config.json is malformed: layer %u has an unknown activation, router or norm", i);
  if (s.mixer == ORION_MIXER_ATTENTION && s.qk_norm != ORION_QK_NORM_PER_HEAD && (s.rope_halves || (s.qkv_bias && !s.keys_as_values) || s.value_gate))
    return set_error(ORION_ERR_MODEL, "layer %u: rotated halves, biases and gates per value come with norms per head", i);
  if (s.mixer == ORION_MIXER_ATTENTION && s.qk_norm == ORION_QK_NORM_PER_HEAD && s.head_gate)
    return set_error(ORION_ERR_MODEL, "layer %u: a gate per head comes with norms over all heads", i);
  if (d_.block == ORION_BLOCK_PARALLEL && (s.experts > 0 || s.ffn_bias))
    return set_error(ORION_ERR_MODEL, "layer %u: a parallel block has a dense feed-forward without biases", i);
  if (d_.block != ORION_BLOCK_PRENORM && (s.activation == ORION_ACT_GEGLU_TANH || s.router == ORION_ROUTER_SOFTMAX || s.router_identity))
    return set_error(ORION_ERR_MODEL, "layer %u: gated dense feed-forwards, corrected routers and identity experts come with prenorm blocks", i);
  if (d_.block == ORION_BLOCK_GATED_POSTNORM && s.mixer == ORION_MIXER_MIN_GRU)
    return set_error(ORION_ERR_MODEL, "layer %u: a gated post-norm block has no min-GRU", i);
  if (s.router == ORION_ROUTER_SOFTMAX_RENORM && d_.block != ORION_BLOCK_GATED_POSTNORM && d_.block != ORION_BLOCK_PRENORM)
    return set_error(ORION_ERR_MODEL, "layer %u: softmax routers come with prenorm and gated post-norm blocks", i);
  return ORION_OK;
}

template <typename T>
int LayeredModel<T>::init() {
  const OrionLayeredDesc &d = d_;
  if (d.hidden_size == 0 || d.vocab_size == 0 || d.num_layers == 0 || d.block > ORION_BLOCK_GATED_POSTNORM || (parallel() && d.conv_taps == 0))
    return set_error(ORION_ERR_MODEL, "config.json is malformed: a model dimension is zero");
  if (d.block_size == 0 || d.max_batch_tokens == 0 || d.max_batch_sequences == 0 || d.num_state_slots == 0)
    return set_error(ORION_ERR_INVALID_REQUEST,
                     "block_size, max_batch_tokens, max_batch_sequences and num_state_slots must be non-zero");
  for (uint32_t i = 0; i < d.num_layers; ++i) ORION_TRY(check_layer(i));
  ORION_TRY(Base::init_step({d.hidden_size, d.vocab_size, d.max_position_embeddings, d.num_blocks, d.block_size, d.max_batch_tokens,
                             d.max_batch_sequences}));
  const size_t H = d.hidden_size;
  if (!gated_postnorm() && (d.learned_positions || d.bigram_buckets))
    return set_error(ORION_ERR_MODEL, "learned positions and pairs of tokens come with gated post-norm blocks");
  if (d.learned_positions && d.max_position_embeddings > d.learned_positions)
    return set_error(ORION_ERR_MODEL, "%u positions asked for, the model has %u", d.max_position_embeddings, d.learned_positions);
  const bool loop = d.loop_times > 0;
  if (loop && (d.block != ORION_BLOCK_PRENORM || d.loop_start >= d.loop_stop || d.loop_stop > d.num_layers))
    return set_error(ORION_ERR_MODEL, "config.json is malformed: layers %u to %u of %u cannot be looped", d.loop_start, d.loop_stop, d.num_layers);
  if (loop) ORION_TRY(alloc(&loop_step_, d.loop_times * H));
  first_run_.resize(d.num_layers);
  auto run = [&](uint32_t i, uint32_t pass) -> int {
    if (pass == 0) {
      first_run_[i] = (uint32_t)layers_.size();
      layers_.emplace_back();
      layers_.back().d = specs_[i];
      ORION_TRY(init_layer(layers_.back()));
    } else {
      const Layer again = layers_[first_run_[i]];
      layers_.push_back(again);
    }
    Layer &L = layers_.back();
    const bool begins = loop && i == d.loop_start;
    L.shift = begins ? loop_step_ + pass * H : nullptr;
    L.restart = begins && pass > 0;
    return init_memory(L);
  };
  for (uint32_t i = 0; i < d.num_layers;) {
    const bool first = loop && i == d.loop_start;
    const uint32_t stop = first ? d.loop_stop : i + 1;
    for (uint32_t pass = 0; pass < (first ? d.loop_times : 1); ++pass)
      for (uint32_t k = i; k < stop; ++k) ORION_TRY(run(k, pass));
    i = stop;
  }
  ORION_TRY(alloc(&embed_, (size_t)d.vocab_size * H));
  if (d.untied_lm_head) ORION_TRY(alloc(&head_, (size_t)d.vocab_size * H));
  if (d.learned_positions) ORION_TRY(alloc(&places_, d.learned_positions * H));
  if (d.bigram_buckets) {
    ORION_TRY(alloc(&pairs_, (d.bigram_buckets + 1) * H));
    ORION_TRY(zeroed(&history_, (size_t)d.num_blocks * d.block_size));
  }
  ORION_TRY(alloc(&final_norm_, H));
  ORION_TRY(init_buffers());
  slots_.resize(num_state_slots());
  ORION_CUDA_CHECK("model init", cudaStreamSynchronize(stream_));
  return ORION_OK;
}

// Rotation tables of a layer, shared by the layers of equal base and size.
template <typename T>
int LayeredModel<T>::init_rope(Layer &L) {
  const OrionLayerDesc &s = L.d;
  const Rope *r = nullptr;
  for (const Rope &x : ropes_)
    if (x.base == s.rope_base && x.dims == s.rope_dims && x.factor == s.yarn_factor && x.original == s.yarn_original && x.fast == s.yarn_fast &&
        x.slow == s.yarn_slow)
      r = &x;
  if (!r) {
    const size_t half = s.rope_dims / 2, positions = d_.max_position_embeddings, n = positions * half;
    std::vector<float> c(n ? n : 1), sn(n ? n : 1);
    std::vector<double> freq(half);
    const double dims = s.rope_dims;
    for (size_t k = 0; k < half; ++k) freq[k] = std::pow(s.rope_base, -2.0 * (double)k / dims);
    double mult = 1.0;
    if (s.yarn_factor > 0) {
      // A pair that turns `fast` times or more within the original length keeps its frequency, one that turns `slow` times or less
      // is stretched by the factor, and those between are blended by their place.
      auto place = [&](double turns) { return dims * std::log(s.yarn_original / (2.0 * M_PI * turns)) / (2.0 * std::log(s.rope_base)); };
      const double lo = std::max(std::floor(place(s.yarn_fast)), 0.0), hi = std::min(std::ceil(place(s.yarn_slow)), dims - 1.0);
      for (size_t k = 0; k < half; ++k) {
        const double ramp = std::min(1.0, std::max(0.0, ((double)k - lo) / std::max(hi - lo, 0.001)));
        freq[k] = freq[k] / s.yarn_factor * ramp + freq[k] * (1.0 - ramp);
      }
      mult = 0.1 * std::log(s.yarn_factor) + 1.0;
    }
    for (size_t p = 0; p < positions; ++p)
      for (size_t k = 0; k < half; ++k) {
        const double angle = (double)p * freq[k];
        c[p * half + k] = (float)(mult * std::cos(angle));
        sn[p * half + k] = (float)(mult * std::sin(angle));
      }
    Rope fresh{s.rope_base, s.yarn_factor, s.yarn_original, s.yarn_fast, s.yarn_slow, s.rope_dims, nullptr, nullptr};
    ORION_TRY(alloc(&fresh.cos, n));
    ORION_TRY(alloc(&fresh.sin, n));
    ORION_CUDA_CHECK("upload rope", cudaMemcpy(fresh.cos, c.data(), n * sizeof(float), cudaMemcpyHostToDevice));
    ORION_CUDA_CHECK("upload rope", cudaMemcpy(fresh.sin, sn.data(), n * sizeof(float), cudaMemcpyHostToDevice));
    ropes_.push_back(fresh);
    r = &ropes_.back();
  }
  L.rope_cos = r->cos, L.rope_sin = r->sin;
  return ORION_OK;
}

// Factors of the queries by position, shared by the layers of equal constants.
template <typename T>
int LayeredModel<T>::init_query_factors(Layer &L) {
  const double coef = L.d.q_temp_coef, every = L.d.q_temp_every;
  if (every == 0) return ORION_OK;
  const QueryFactors *known = nullptr;
  for (const QueryFactors &q : query_factors_)
    if (q.coef == coef && q.every == every) known = &q;
  if (!known) {
    std::vector<float> f(d_.max_position_embeddings);
    for (size_t p = 0; p < f.size(); ++p) f[p] = (float)(1.0 + coef * std::log(std::floor(((double)p + 1.0) / every) + 1.0));
    QueryFactors fresh{coef, every, nullptr};
    ORION_TRY(alloc(&fresh.table, f.size()));
    ORION_CUDA_CHECK("upload query factors", cudaMemcpy(fresh.table, f.data(), f.size() * sizeof(float), cudaMemcpyHostToDevice));
    query_factors_.push_back(fresh);
    known = &query_factors_.back();
  }
  L.in.q_factor = known->table;
  return ORION_OK;
}

template <typename T>
int LayeredModel<T>::init_layer(Layer &L) {
  const OrionLayeredDesc &d = d_;
  const OrionLayerDesc &s = L.d;
  const size_t H = d.hidden_size;
  ORION_TRY(alloc(&L.norm, H));
  if (sandwich()) ORION_TRY(alloc(&L.norm_post, H));
  if (parallel()) ORION_TRY(alloc(&L.conv1, H * d.conv_taps));
  if (L.latent()) {
    L.ls = LatentShape{s.heads, s.dim, s.rot_dim, s.value_dim, s.kv_rank, s.window, s.rope_dims, d.block_size,
                       odd_groups(s.kv_rank + s.rot_dim), (float)s.scale, (float)d.norm_eps, !s.ungated};
    L.mix_in = L.ls.cols(), L.mix_out = L.ls.out_cols();
    ORION_TRY(alloc(&L.latent_norm, s.kv_rank));
    ORION_TRY(alloc(&L.w_uk, (size_t)s.heads * (s.dim + s.value_dim) * s.kv_rank));  // one matrix for the expansion of prompts
    L.w_uv = L.w_uk + (size_t)s.heads * s.dim * s.kv_rank;
    ORION_TRY(init_rope(L));
  } else if (L.attention()) {
    // [q | k | v | gate], the rows of the matrix padded so that the partial sums of a row start on 32 bytes
    const uint32_t qkv = s.heads * s.dim + s.kv_heads * (s.dim + (s.keys_as_values ? 0 : s.value_dim));
    L.mix_in = pad8(qkv + (s.head_gate ? s.heads : 0) + (s.value_gate ? s.heads * s.value_dim : 0));
    L.mix_out = s.heads * s.value_dim;
    ORION_TRY(init_rope(L));
    if (s.qk_norm) {
      const bool own = s.qk_norm == ORION_QK_NORM_PER_HEAD;
      ORION_TRY(alloc(&L.q_norm, (size_t)(own ? 1 : s.heads) * s.dim));
      ORION_TRY(alloc(&L.k_norm, (size_t)(own ? 1 : s.kv_heads) * s.dim));
    }
    if (s.qkv_bias) ORION_TRY(alloc(&L.mix_bias, qkv));
    if (s.sinks) ORION_TRY(zeroed(&L.sinks, s.heads));
    if (s.keys_as_values) ORION_TRY(alloc(&L.q_gain, (size_t)s.heads * s.dim));
    if (s.distance_bias) {
      ORION_TRY(alloc(&L.dist_mult, s.heads));
      ORION_TRY(alloc(&L.dist_rate, s.heads));
    }
    // 16-bit caches pad the heads to sizes of the tensor-core kernels where those cover them
    const uint32_t dk = DTypeOf<T>::is_bf16 ? attention_padded_dim(s.dim, s.value_dim) : 0;
    const uint32_t dv = DTypeOf<T>::is_bf16 ? attention_padded_dim(s.value_dim, s.dim) : 0;
    L.kv = KvLayout{1, d.num_blocks, s.kv_heads, d.block_size, dk ? dk : s.dim, dk ? 1u : 0u, dk ? dv : s.value_dim,
                    s.keys_as_values ? (uint32_t)(sizeof(float) / sizeof(T)) : 0};
    L.tuned = DTypeOf<T>::is_bf16 && attention_form_supported(L.kv, s.heads);
    L.in = AttnInputs{s.heads, s.kv_heads, s.dim, s.value_dim, s.rope_dims, L.mix_in, (float)d.norm_eps, s.keys_as_values ? L.q_gain : L.q_norm, L.k_norm, L.rope_cos, L.rope_sin,
                      s.qk_norm == ORION_QK_NORM_PER_HEAD, s.rope_halves != 0, L.mix_bias, s.keys_as_values != 0};
    ORION_TRY(init_query_factors(L));
    L.form.scale = (float)s.scale;
    L.form.softcap = (float)s.softcap;
    L.form.range = KeyRange{s.window, s.chunk, s.keep_first};
    L.form.sinks = L.sinks;
    L.form.dist_mult = L.dist_mult, L.form.dist_rate = L.dist_rate;
    L.form.out_dim = s.value_dim;
    if (L.tuned) {
      const uint32_t positions = 128 / (s.heads / s.kv_heads);
      bool known = false;
      for (const TileSet &t : tile_sets_) known |= t.positions == positions;
      if (!known) tile_sets_.push_back(TileSet{positions, 0, 0});
    }
  } else if (L.linear()) {
    L.gla = GlaShape{s.heads, s.dim, s.value_dim, s.decay_rank, 0, (float)s.decay_tau, (float)d.norm_eps};
    L.mix_in = L.gla.ld = pad8(L.gla.cols());
    L.mix_out = L.gla.v_cols();
    ORION_TRY(alloc(&L.w_decay, (size_t)L.gla.q_cols() * s.decay_rank));
    ORION_TRY(alloc(&L.mix_bias, L.gla.q_cols()));
    ORION_TRY(alloc(&L.out_norm, s.value_dim));
  } else {
    L.mix_in = 3 * s.width, L.mix_out = s.width;
    ORION_TRY(alloc(&L.mix_bias, 2 * (size_t)s.width));
  }
  if (gated_postnorm()) {
    L.gate_at = pad8(L.mix_in);
    L.mix_in = pad8(L.gate_at + d.hidden_size);
    L.ls.ld = L.in.ld = L.gla.ld = L.mix_in;
    ORION_TRY(alloc(&L.gate_bias, H));
  }
  ORION_TRY(zeroed(&L.w_mix, (size_t)L.mix_in * H));
  // Activations start at multiples of 8 columns; the weights of the columns between them are zero.
  L.ff_at = parallel() ? pad8(L.mix_out) : 0;
  L.cat = parallel() ? L.ff_at + pad8(s.ffn_dim) : pad8(L.mix_out);
  L.ff_ld = parallel() ? L.cat : pad8(s.ffn_dim);
  if (L.attention()) L.form.ldo = L.cat;
  ORION_TRY(zeroed(&L.w_out, H * L.cat));
  if (!L.has_ffn()) return ORION_OK;
  if (parallel()) ORION_TRY(alloc(&L.conv2, H * d.conv_taps));
  else ORION_TRY(alloc(&L.norm2, H));
  if (sandwich()) ORION_TRY(alloc(&L.norm2_post, H));
  if (gated_postnorm()) ORION_TRY(alloc(&L.ff_gate_bias, H));
  if (s.experts > 0) {
    L.moe = MoeShape{d.hidden_size, s.experts, s.experts_per_token, s.ffn_dim, s.shared_dim, s.router_identity};
    L.moe.softmax = L.moe.weigh_output = s.router != ORION_ROUTER_SIGMOID_INPUT;
    L.moe.renorm = s.router == ORION_ROUTER_SOFTMAX_RENORM;
    L.moe.groups = s.router_groups, L.moe.keep = s.router_keep;
    const GatedKind kind = s.expert_form == ORION_EXPERT_CLAMPED ? kGatedClamped : (s.expert_form == ORION_EXPERT_GELU ? kPlainGelu : kGatedSilu);
    L.moe.act = GatedAct{kind, (float)s.expert_limit}, L.moe.shared_act = GatedAct{kind, (float)s.shared_limit};
    if (gated_postnorm()) {
      L.ff_gate_at = pad8(L.moe.outputs());
      L.moe.logits_ld = pad8(L.ff_gate_at + d.hidden_size);
    }
    ORION_TRY(zeroed(&L.w_router, (size_t)L.moe.row_ld() * H));
    if (s.router == ORION_ROUTER_SOFTMAX) ORION_TRY(alloc(&L.correction, L.moe.outputs()));
    ORION_TRY(alloc(&L.e_up, (size_t)s.experts * L.moe.up_cols() * H));
    ORION_TRY(alloc(&L.e_down, (size_t)s.experts * H * s.ffn_dim));
    if (s.shared_dim) {
      ORION_TRY(alloc(&L.s_up, (size_t)L.moe.shared_up_cols() * H));
      ORION_TRY(alloc(&L.s_down, H * s.shared_dim));
    }
    return ORION_OK;
  }
  if (gated_postnorm()) ORION_TRY(alloc(&L.w_ff_gate, H * H));
  ORION_TRY(alloc(&L.w_up, (size_t)(L.gated_ffn() ? 2 : 1) * s.ffn_dim * H));
  if (!parallel()) ORION_TRY(zeroed(&L.w_down, H * L.ff_ld));
  if (s.ffn_bias) {
    ORION_TRY(alloc(&L.up_bias, s.ffn_dim));
    ORION_TRY(alloc(&L.down_bias, H));
  }
  return ORION_OK;
}

template <typename T>
int LayeredModel<T>::init_memory(Layer &L) {
  const size_t copies = 2 * (size_t)d_.num_state_slots, keep = d_.conv_taps ? d_.conv_taps - 1 : 0;
  if (parallel()) ORION_TRY(zeroed(&L.conv_state, copies * keep * d_.hidden_size));
  if (L.linear()) ORION_TRY(zeroed(&L.rec_state, copies * L.gla.state_floats()));
  if (L.d.mixer == ORION_MIXER_MIN_GRU) ORION_TRY(zeroed(&L.rec_state, copies * L.d.width));
  if (L.cache_elems()) ORION_TRY(zeroed(&L.cache, d_.num_blocks * L.cache_elems()));
  return ORION_OK;
}

// Work buffers, sized for the largest batch of any layer.
template <typename T>
int LayeredModel<T>::init_buffers() {
  constexpr bool kBf16 = DTypeOf<T>::is_bf16;
  const OrionLayeredDesc &d = d_;
  const size_t H = d.hidden_size, rows = d.max_batch_tokens;
  const uint32_t few = (uint32_t)std::min<uint64_t>(rows, (uint64_t)kFewRows * d.max_batch_sequences);
  size_t cat = 0, qcols = 0, gates = 0, value_gates = 0, qa = 0;
  struct { size_t choices = 0, histogram = 0, tiles = 0, x = 0, act = 0, up = 0, down = 0; } moe;
  auto grow = [](size_t &a, size_t b) { a = std::max(a, b); };
  for (const Layer &L : layers_) {
    const OrionLayerDesc &s = L.d;
    grow(cat, L.cat);
    const std::pair<uint32_t, uint32_t> products[] = {
        {L.mix_in, (uint32_t)H}, {(uint32_t)H, L.cat}, {s.experts ? L.moe.row_ld() : (L.gated_ffn() ? 2 : 1) * s.ffn_dim, (uint32_t)H}, {L.w_down ? (uint32_t)H : 0, L.ff_ld},
        {L.w_ff_gate ? (uint32_t)H : 0, (uint32_t)H}};
    for (const auto &[n, k] : products)
      if (n) grow(partial_floats_, gemm_partial_floats(kBf16, (uint32_t)rows, n, k));
    if (L.w_down) grow(cat, L.ff_ld);
    if (L.latent()) grow(qcols, L.ls.q_cols());
    if (L.attention()) {
      grow(qcols, (size_t)s.heads * L.kv.head_dim);
      if (s.head_gate) grow(gates, s.heads);
      if (s.value_gate) grow(value_gates, (size_t)s.heads * s.value_dim);
    }
    if (tuned(L)) grow(qa, (size_t)few * s.heads * L.ls.kv_cols());
    for (uint32_t r = 1; r <= few; ++r) {
      if (tuned(L)) grow(scratch_floats_, latent_decode_scratch_floats(L.ls, r, latent_decode_splits(L.ls, r, d.max_position_embeddings)));
      if (L.tuned)
        grow(scratch_floats_, decode_scratch_floats(r, s.heads, L.kv.v_dim(), decode_form_splits(L.kv, s.heads, r, L.form.range.most(d.max_position_embeddings - 1))));
    }
    if (s.experts) {
      // k splits come with small batches only
      for (uint32_t r = 1; r <= rows; r = r < 64 ? r + 1 : (r < rows ? (uint32_t)rows : (uint32_t)rows + 1)) {
        const MoePlan p = moe_plan(kBf16, L.moe, r);
        const size_t choices = (size_t)r * L.moe.top;
        grow(moe.choices, choices), grow(moe.histogram, moe_histogram_words(L.moe, r));
        grow(moe.x, choices * H), grow(moe.act, choices * s.ffn_dim + (size_t)r * s.shared_dim);
        grow(moe.up, moe_up_floats(kBf16, L.moe, r)), grow(moe.down, p.down_splits * choices * H);
        grow(partial_floats_, p.down_splits * (size_t)r * H);
      }
      for (uint32_t r = 1; r <= rows; ++r) grow(moe.tiles, moe_plan(kBf16, L.moe, r).tiles);
    }
  }
  ORION_TRY(alloc(&partial_, partial_floats_));
  if (gated_postnorm()) ORION_TRY(alloc(&out_partial_, partial_floats_));
  if (parallel()) {
    ORION_TRY(alloc(&conv_m_, rows * H));
    ORION_TRY(alloc(&conv_f_, rows * H));
  }
  ORION_TRY(zeroed(&cat_, rows * cat));  // columns that nobody writes meet zero weights and must be finite
  ORION_TRY(zeroed(&qbuf_, rows * qcols));  // so must the padding of queries, which meets that of the keys
  ORION_TRY(alloc(&gate_, rows * gates));
  ORION_TRY(alloc(&value_gate_, rows * value_gates));
  ORION_TRY(alloc(&qa_, qa));
  ORION_TRY(zeroed(&scratch_, scratch_floats_));
  if (moe.choices) {
    ORION_TRY(alloc(&moe_.chosen, moe.choices));
    ORION_TRY(alloc(&moe_.score, moe.choices));
    ORION_TRY(alloc(&moe_.place, moe.choices));
    ORION_TRY(alloc(&moe_.row_score, moe.choices));
    ORION_TRY(alloc(&moe_.histogram, moe.histogram));
    ORION_TRY(alloc(&moe_.tiles, moe.tiles));
    ORION_TRY(zeroed(&moe_.x, moe.x));
    ORION_TRY(zeroed(&moe_.act, moe.act));
    ORION_TRY(alloc(&moe_.up, moe.up));
    ORION_TRY(alloc(&moe_.down, moe.down));
  }
  return ORION_OK;
}

template <typename T>
bool LayeredModel<T>::place(const std::string &name, Place *p) const {
  const uint64_t H = d_.hidden_size;
  auto matrix = [&](T *dst, uint64_t rows, uint64_t cols, uint64_t ld = 0) {
    p->dst = dst, p->rows = rows, p->cols = cols, p->ld = ld ? ld : cols, p->matrix = true;
    return dst != nullptr && rows > 0;
  };
  auto filters = [&](T *dst) {
    p->transposed = true;
    return matrix(dst, H, d_.conv_taps);
  };
  auto vector = [&](float *dst, uint64_t n, float fill = 1.0f) {
    p->vec = dst, p->rows = 1, p->cols = n, p->matrix = false, p->fill = fill;
    return dst != nullptr && n > 0;
  };
  if (name == "loop.step") {
    vector(loop_step_, H, 0.0f);
    p->rows = d_.loop_times, p->matrix = true;
    return loop_step_ != nullptr;
  }
  auto gain = [&](float *dst) {  // of a norm of the residual stream
    if (!d_.scalar_norms) return vector(dst, H);
    p->copies = H;
    return vector(dst, 1);
  };
  if (name == "embed") return matrix(embed_, d_.vocab_size, H);
  if (name == "bigram") return matrix(pairs_, d_.bigram_buckets + 1, H);
  if (name == "pos") return matrix(places_, d_.learned_positions, H);
  if (name == "head") return matrix(head_, d_.vocab_size, H);
  if (name == "final.norm") return gain(final_norm_);
  unsigned i = 0;
  int used = 0;
  if (sscanf(name.c_str(), "l%u.%n", &i, &used) != 1 || used == 0 || i >= first_run_.size()) return false;
  const std::string rest = name.substr((size_t)used);
  const Layer &L = layers_[first_run_[i]];
  const OrionLayerDesc &s = L.d;
  if (rest == "norm1") return gain(L.norm);
  if (rest == "norm1b") return gain(L.norm_post);
  if (rest == "norm2") return gain(L.norm2);
  if (rest == "norm2b") return gain(L.norm2_post);
  if (rest == "rg1") return gated_postnorm() && matrix(L.w_mix + (uint64_t)L.gate_at * H, H, H);
  if (rest == "rg2") return gated_postnorm() && matrix(L.w_router ? L.w_router + (uint64_t)L.ff_gate_at * H : L.w_ff_gate, H, H);
  if (rest == "rg1.b") return vector(L.gate_bias, H, 0.0f);
  if (rest == "rg2.b") return vector(L.ff_gate_bias, H, 0.0f);
  if (rest == "canon1") return L.conv1 && filters(L.conv1);
  if (rest == "canon2") return L.conv2 && filters(L.conv2);
  if (rest.compare(0, 4, "mlp.") == 0) {
    const std::string t = rest.substr(4);
    // an expert's gate and up rows alternate in one matrix
    const bool plain = s.experts > 0 && L.moe.act.plain();
    auto expert = [&](const std::string &part, T *up, T *down, uint64_t ffn) {
      if (plain && part == "gate") return false;
      if (plain && part == "up") return matrix(up, ffn, H);
      if (part == "gate") return matrix(up, ffn, H, 2 * H);
      if (part == "up") return matrix(up ? up + H : nullptr, ffn, H, 2 * H);
      if (part == "down") return matrix(down, H, ffn);
      return false;
    };
    if (t == "router") return matrix(L.w_router, L.moe.outputs(), H);
    if (t == "correction") return vector(L.correction, L.moe.outputs(), 0.0f);
    if (t.compare(0, 7, "shared.") == 0) return expert(t.substr(7), L.s_up, L.s_down, s.shared_dim);
    unsigned e = 0;
    int at = 0;
    if (sscanf(t.c_str(), "e%u.%n", &e, &at) == 1 && at > 0) {
      if (e >= s.experts) return false;
      return expert(t.substr((size_t)at), L.e_up + (uint64_t)e * L.moe.up_cols() * H, L.e_down + e * H * s.ffn_dim, s.ffn_dim);
    }
    if (s.experts > 0 || !L.has_ffn()) return false;
    if (L.gated_ffn() && t != "down") return expert(t, L.w_up, nullptr, s.ffn_dim);
    if (t == "up") return matrix(L.w_up, s.ffn_dim, H);
    if (t == "down") return parallel() ? matrix(L.w_out + L.ff_at, H, s.ffn_dim, L.cat) : matrix(L.w_down, H, s.ffn_dim, L.ff_ld);
    if (t == "up.b") return vector(L.up_bias, s.ffn_dim, 0.0f);
    if (t == "down.b") return vector(L.down_bias, H, 0.0f);
    return false;
  }
  if (rest.compare(0, 4, "mix.") != 0) return false;
  const std::string t = rest.substr(4);
  if (t == "o") return matrix(L.w_out, H, L.mix_out, L.cat);
  if (L.attention()) {
    const uint64_t nq = (uint64_t)s.heads * s.dim, nk = (uint64_t)s.kv_heads * s.dim, nv = (uint64_t)s.kv_heads * s.value_dim;
    if (t == "q") return matrix(L.w_mix, nq, H);
    if (t == "k") return matrix(L.w_mix + nq * H, nk, H);
    if (t == "v") return !s.keys_as_values && matrix(L.w_mix + (nq + nk) * H, nv, H);
    if (t == "r1") return vector(L.dist_mult, s.heads, 0.5f);
    if (t == "r2") return vector(L.dist_rate, s.heads, 0.1f);
    if (t == "g") return (s.head_gate || s.value_gate) && matrix(L.w_mix + (nq + nk + nv) * H, s.value_gate ? s.heads * s.value_dim : s.heads, H);
    const bool own = s.qk_norm == ORION_QK_NORM_PER_HEAD;
    if (t == "q.norm") return vector(L.q_norm, own ? s.dim : nq);
    if (t == "k.norm") return vector(L.k_norm, own ? s.dim : nk);
    if (t == "q.b") return vector(L.mix_bias, nq, 0.0f);
    if (t == "k.b") return vector(L.mix_bias ? L.mix_bias + nq : nullptr, nk, 0.0f);
    if (t == "v.b") return !s.keys_as_values && vector(L.mix_bias ? L.mix_bias + nq + nk : nullptr, nv, 0.0f);
    if (t == "sink") return s.sinks == ORION_SINK_LEARNED && vector(L.sinks, s.heads, 0.0f);
    return false;
  }
  if (L.latent()) {
    const LatentShape &a = L.ls;
    if (t == "q") return matrix(L.w_mix, a.q_cols(), H);
    if (t == "dkv") return matrix(L.w_mix + a.q_cols() * H, a.kv_cols(), H);
    if (t == "g") return a.gated && matrix(L.w_mix + (a.q_cols() + a.kv_cols()) * H, a.out_cols(), H);
    if (t == "dkv.norm") return vector(L.latent_norm, s.kv_rank);
    if (t == "uk") return matrix(L.w_uk, (uint64_t)s.heads * s.dim, s.kv_rank);
    if (t == "uv") return matrix(L.w_uv, (uint64_t)s.heads * s.value_dim, s.kv_rank);
    return false;
  }
  if (L.linear()) {
    const uint64_t nq = L.gla.q_cols(), nv = L.gla.v_cols();
    if (t == "q") return matrix(L.w_mix, nq, H);
    if (t == "k") return matrix(L.w_mix + nq * H, nq, H);
    if (t == "v") return matrix(L.w_mix + 2 * nq * H, nv, H);
    if (t == "g") return matrix(L.w_mix + (2 * nq + nv) * H, nv, H);
    if (t == "a1") return matrix(L.w_mix + (2 * nq + 2 * nv) * H, s.decay_rank, H);
    if (t == "a2") return matrix(L.w_decay, nq, s.decay_rank);
    if (t == "a2.b") return vector(L.mix_bias, nq, 3.0f);  // a randomly initialised model forgets slowly
    if (t == "norm") return vector(L.out_norm, s.value_dim);
    return false;
  }
  if (t == "z") return matrix(L.w_mix, s.width, H);
  if (t == "x") return matrix(L.w_mix + s.width * H, s.width, H);
  if (t == "g") return matrix(L.w_mix + 2 * (uint64_t)s.width * H, s.width, H);
  if (t == "z.b") return vector(L.mix_bias, s.width, 0.0f);
  if (t == "x.b") return vector(L.mix_bias + s.width, s.width, 0.0f);
  return false;
}

template <typename T>
std::vector<std::string> LayeredModel<T>::tensor_names() const {
  std::vector<std::string> names;
  auto add = [&](const std::string &name) {
    if (uses_tensor(name.c_str())) names.push_back(name);
  };
  for (const char *n : {"embed", "head", "final.norm", "loop.step", "bigram", "pos"}) add(n);
  for (uint32_t i = 0; i < d_.num_layers; ++i) {
    const std::string l = "l" + std::to_string(i) + ".";
    for (const char *rest : {"norm1", "norm1b", "norm2", "norm2b", "canon1", "canon2", "mlp.up", "mlp.up.b", "mlp.down", "mlp.down.b", "mlp.router",
                             "mlp.shared.gate", "mlp.shared.up", "mlp.shared.down", "mix.o", "mix.q", "mix.k", "mix.v", "mix.q.norm", "mix.k.norm",
                             "mix.sink", "mix.dkv", "mix.dkv.norm", "mix.uk", "mix.uv", "mix.g", "mix.z", "mix.x", "mix.z.b", "mix.x.b", "mlp.gate", "mlp.correction", "mix.q.b", "mix.k.b", "mix.v.b", "mix.norm", "mix.a1",
                             "mix.a2", "mix.a2.b", "rg1", "rg1.b", "rg2", "rg2.b", "mix.r1", "mix.r2"})
      add(l + rest);
    for (uint32_t e = 0; e < specs_[i].experts; ++e)
      for (const char *part : {".gate", ".up", ".down"}) add(l + "mlp.e" + std::to_string(e) + part);
  }
  return names;
}

template <typename T>
int LayeredModel<T>::load_tensor(const char *name, int dtype, const uint64_t *shape, int ndim, const void *data) {
  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  if (dtype_size(dtype) == 0) return set_error(ORION_ERR_MODEL, "unsupported dtype %d (tensor `%s`)", dtype, name);
  if (!data || ndim < 0 || ndim > 2) return set_error(ORION_ERR_MODEL, "tensor `%s` has rank %d", name, ndim);
  Place p;
  if (!place(name, &p)) return set_error(ORION_ERR_MODEL, "tensor `%s` is not part of the model", name);
  const uint64_t R = ndim == 2 ? shape[0] : 1, C = ndim == 0 ? 1 : shape[ndim - 1];
  if (R != p.rows || C != p.cols || (ndim == 2) != p.matrix)
    return set_error(ORION_ERR_MODEL, "tensor `%s` has shape [%llu, %llu], expected [%llu, %llu]", name, (unsigned long long)R,
                     (unsigned long long)C, (unsigned long long)p.rows, (unsigned long long)p.cols);
  finalized_ = false;
  if (p.vec) {
    ORION_TRY(upload_slice(nullptr, p.vec, data, dtype, C, 0, R, 0, C));
    if (p.copies) {
      float value = 0.f;
      ORION_CUDA_CHECK("upload tensor", cudaMemcpy(&value, p.vec, sizeof(float), cudaMemcpyDeviceToHost));
      ORION_TRY(set_constant(p.vec, p.copies, value));
    }
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
  std::vector<std::string> got(got_);
  std::sort(got.begin(), got.end());
  for (const std::string &n : tensor_names())
    if (!std::binary_search(got.begin(), got.end(), n)) return set_error(ORION_ERR_MODEL, "missing tensor `%s`", n.c_str());
  for (Layer &L : layers_) {
    if (!L.q_gain) continue;
    const size_t nq = (size_t)L.d.heads * L.d.dim, nk = (size_t)L.d.kv_heads * L.d.dim, group = L.d.heads / L.d.kv_heads;
    std::vector<float> q(nq), k(nk);
    ORION_CUDA_CHECK("gains", cudaMemcpy(q.data(), L.q_norm, nq * sizeof(float), cudaMemcpyDeviceToHost));
    ORION_CUDA_CHECK("gains", cudaMemcpy(k.data(), L.k_norm, nk * sizeof(float), cudaMemcpyDeviceToHost));
    for (size_t i = 0; i < nq; ++i) q[i] *= k[i / L.d.dim / group * L.d.dim + i % L.d.dim];
    ORION_CUDA_CHECK("gains", cudaMemcpy(L.q_gain, q.data(), nq * sizeof(float), cudaMemcpyHostToDevice));
  }
  lm_head_ = head_ ? head_ : embed_;
  finalized_ = true;
  return ORION_OK;
}

template <typename T>
int LayeredModel<T>::init_random(uint64_t seed, float std) {
  // N(0, std) matrices, norm gains 1, zero biases and sinks; the filters keep most of the current row's weight out of
  // the sum like a trained one would (std 0.1 per tap).
  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  for (const std::string &n : tensor_names()) {
    Place p;
    place(n, &p);
    if (p.vec) {
      ORION_TRY(set_constant(p.vec, p.copies ? p.copies : p.rows * p.cols, p.fill));
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
  const bool state = has_state();
  if (state && (!b.state_slots || b.num_state_slots != S))
    return set_error(ORION_ERR_INVALID_REQUEST, "this model needs a state slot for each of the %llu sequences", (unsigned long long)S);
  std::vector<bool> taken(slots_.size(), false);
  uint64_t row = 0;
  for (uint64_t s = 0; s < S; ++s) {
    const uint64_t n = b.slot_token_counts[s];
    if (n == 0) return set_error(ORION_ERR_INTERNAL, "a scheduled sequence contributed zero tokens");
    for (uint64_t i = 1; i < n; ++i)
      if (b.positions[row + i] != b.positions[row] + i)
        return set_error(ORION_ERR_INTERNAL, "the positions of sequence %llu are not consecutive", (unsigned long long)s);
    if (state) {
      const uint32_t slot = b.state_slots[s];
      if (slot >= slots_.size())
        return set_error(ORION_ERR_INTERNAL, "state slot %u out of range (have %zu)", slot, slots_.size());
      if (taken[slot]) return set_error(ORION_ERR_INTERNAL, "state slot %u is named twice in one batch", slot);
      taken[slot] = true;
      if (b.positions[row] != 0 && (!slots_[slot].live || slots_[slot].tokens != b.positions[row]))
        return set_error(ORION_ERR_INTERNAL, "sequence %llu goes on at position %u but its state covers %llu tokens",
                         (unsigned long long)s, b.positions[row], (unsigned long long)(slots_[slot].live ? slots_[slot].tokens : 0));
    }
    row += n;
  }
  return ORION_OK;
}

template <typename T>
void LayeredModel<T>::fill_extra(const BatchView &b, uint32_t *w) {
  const uint64_t S = b.num_sequences;
  uint32_t *first = w, *read = w + S + 1, *write = read + S, *few = write + S;
  uint64_t row = 0;
  few_rows_ = portions_ = gla_chunks_ = gla_portions_ = 0;
  for (TileSet &t : tile_sets_) t.count = 0;
  for (uint64_t s = 0; s < S; ++s) {
    first[s] = (uint32_t)row;
    read[s] = write[s] = kNoState;
    if (has_state()) {
      const uint32_t slot = b.state_slots[s], copy = slots_[slot].copy;
      if (b.positions[row] != 0) read[s] = 2 * slot + copy;
      write[s] = 2 * slot + (copy ^ 1u);
    }
    if (b.slot_token_counts[s] <= kFewRows)
      for (uint64_t i = 0; i < b.slot_token_counts[s]; ++i) few[few_rows_++] = (uint32_t)(row + i);
    row += b.slot_token_counts[s];
  }
  first[S] = (uint32_t)row;
}

template <typename T>
int LayeredModel<T>::fill_tiles(const BatchView &b, uint32_t *t, typename Base::Meta &mt) {
  ORION_TRY(fill_latent_tiles(b, t, mt));
  size_t at = 4 * (2 * (size_t)b.num_sequences + b.num_tokens / kLatentTileRows + 1);
  for (TileSet &set : tile_sets_) {
    set.offset = at;
    auto *tiles = reinterpret_cast<PrefillTile *>(t + at);
    uint64_t row = 0;
    for (uint64_t s = 0; s < b.num_sequences; ++s) {
      const uint64_t n = b.slot_token_counts[s];
      for (uint64_t i = 0; n > kFewRows && i < n; i += set.positions) {
        const uint32_t rows = (uint32_t)std::min<uint64_t>(set.positions, n - i);
        tiles[set.count++] = PrefillTile{(uint32_t)(row + i), rows, (uint32_t)s, b.positions[row + i] + rows - 1};
      }
      row += n;
    }
    at += 4 * ((size_t)b.num_sequences + b.num_tokens / set.positions + 1);
  }
  return fill_gla_chunks(b, t, at);
}

// The sequences that bring more than a few rows, cut into chunks, and scratch for the largest of the layers that take them.
template <typename T>
int LayeredModel<T>::fill_gla_chunks(const BatchView &b, uint32_t *t, size_t at) {
  if (!DTypeOf<T>::is_bf16) return ORION_OK;
  gla_at_ = at;
  auto *portions = reinterpret_cast<GlaPortion *>(t + at);
  auto *chunks = reinterpret_cast<GlaChunk *>(t + at + 4 * b.num_sequences);
  uint64_t row = 0;
  for (uint64_t s = 0; s < b.num_sequences; ++s) {
    const uint64_t n = b.slot_token_counts[s];
    if (n > kFewRows) {
      portions[gla_portions_++] = GlaPortion{(uint32_t)s, gla_chunks_, (uint32_t)((n + kGlaChunk - 1) / kGlaChunk), 0};
      for (uint64_t i = 0; i < n; i += kGlaChunk)
        chunks[gla_chunks_++] = GlaChunk{(uint32_t)(row + i), (uint32_t)std::min<uint64_t>(kGlaChunk, n - i), 0, 0};
    }
    row += n;
  }
  size_t need = 0;
  for (const Layer &L : layers_)
    if (L.linear() && gla_chunks_ > 0 && gla_chunks_supported(L.gla)) need = std::max(need, gla_scratch_bytes(L.gla, gla_chunks_, (uint32_t)b.num_tokens));
  if (need > gla_scratch_bytes_) {
    if (gla_scratch_) cudaFree(gla_scratch_);  // the previous step has ended
    gla_scratch_ = nullptr, gla_scratch_bytes_ = 0;
    ORION_CUDA_CHECK("allocate chunk operands", cudaMalloc(&gla_scratch_, need + need / 4));
    gla_scratch_bytes_ = need + need / 4;
  }
  return ORION_OK;
}

// Portions and tiles of the sequences that bring more than a few rows, and room for their expanded rows.
template <typename T>
int LayeredModel<T>::fill_latent_tiles(const BatchView &b, uint32_t *t, typename Base::Meta &mt) {
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
  if (!has_state()) return;
  for (uint64_t s = 0; s < b.num_sequences; ++s) {
    Slot &x = slots_[b.state_slots[s]];
    x.tokens = (uint64_t)b.positions[row] + b.slot_token_counts[s];
    x.copy ^= 1u;
    x.live = true;
    row += b.slot_token_counts[s];
  }
}

template <typename T>
int LayeredModel<T>::poll_errors() {
  ORION_TRY(Base::poll_errors());
  if (!DTypeOf<T>::is_bf16) return ORION_OK;
  bool latent = false, attention = false, experts = false, linear = false;
  for (const Layer &L : layers_) latent |= L.latent(), attention |= L.attention(), experts |= L.moe.experts > 0, linear |= L.linear();
  uint32_t code = 0;
  auto poll = [&](int (*read)(uint32_t *), const char *what) -> int {
    ORION_TRY(read(&code));
    if (code) return set_error(ORION_ERR_BACKEND, "backend cuda failed at %s: a bounded pipeline wait ran out (code %u)", what, code);
    return ORION_OK;
  };
  if (latent) {
    ORION_TRY(poll(latent_poll_error, "latent attention"));
    ORION_TRY(poll(latent_prefill_poll_error, "latent attention"));
  }
  if (attention) {
    ORION_TRY(poll(decode_poll_error, "attention"));
    ORION_TRY(poll(prefill_tc_poll_error, "prefill attention"));
  }
  if (experts) ORION_TRY(poll(moe_poll_error, "mixture of experts"));
  if (linear) ORION_TRY(poll(gla_poll_error, "gated linear attention"));
  return ORION_OK;
}

template <typename T>
int LayeredModel<T>::fill_kv_random(uint64_t seed, float std) {
  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  for (const Layer &L : layers_)
    if (L.cache) {
      ORION_TRY(fill_random(L.cache, d_.num_blocks * L.cache_elems(), seed, std));
      if (L.attention() && L.kv.factor_elems) ORION_TRY(launch_fill_factors<T>(L.cache, L.kv, 1.f, stream_));
    }
  ORION_CUDA_CHECK("fill_kv_random", cudaStreamSynchronize(stream_));
  return ORION_OK;
}

// The caches of the attention layers, one after the other: latents as [block][slot][kv_rank + rot_dim], keys and then values as
// [block][kv head][slot][dim], where the values are the keys one set of rows and then the factors of the keys.
template <typename T>
int LayeredModel<T>::read_kv(float *out, uint64_t capacity) {
  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  const size_t tokens = (size_t)d_.num_blocks * d_.block_size;
  for (const Layer &L : layers_) {
    if (!L.cache) continue;
    const size_t cols = L.latent() ? L.ls.kv_cols() : L.d.kv_heads * (L.d.dim + (L.d.keys_as_values ? 1 : L.d.value_dim));
    const size_t stride = L.latent() ? L.ls.row_stride : cols, n = tokens * stride;
    if (capacity < tokens * cols) return set_error(ORION_ERR_INVALID_REQUEST, "KV read-back buffer is too small");
    ORION_TRY(ensure_stage(&stage_f32_, &stage_f32_cap_, n * sizeof(float)));
    float *tmp = static_cast<float *>(stage_f32_);
    if (L.latent()) ORION_TRY(launch_convert_to_f32<T>(L.cache, tmp, n, stream_));
    else ORION_TRY(launch_arena_rows<T>(L.cache, L.kv, L.d.dim, L.d.value_dim, tmp, stream_));
    ORION_CUDA_CHECK("read_kv", cudaMemcpy2DAsync(out, cols * sizeof(float), tmp, stride * sizeof(float), cols * sizeof(float), tokens,
                                                  cudaMemcpyDeviceToHost, stream_));
    ORION_CUDA_CHECK("read_kv", cudaStreamSynchronize(stream_));
    out += tokens * cols;
    capacity -= tokens * cols;
  }
  return ORION_OK;
}

#define ORION_INSTANTIATE(T)                                                                                             \
  template int LayeredModel<T>::init();                                                                                  \
  template bool LayeredModel<T>::place(const std::string &, Place *) const;                                              \
  template int LayeredModel<T>::load_tensor(const char *, int, const uint64_t *, int, const void *);                     \
  template int LayeredModel<T>::init_random(uint64_t, float);                                                            \
  template int LayeredModel<T>::finalize();                                                                              \
  template int LayeredModel<T>::fill_kv_random(uint64_t, float);                                                         \
  template int LayeredModel<T>::read_kv(float *, uint64_t);                                                              \
  template int LayeredModel<T>::check_batch(const BatchView &);                                                          \
  template void LayeredModel<T>::fill_extra(const BatchView &, uint32_t *);                                              \
  template int LayeredModel<T>::fill_tiles(const BatchView &, uint32_t *, StepModel<T>::Meta &);                         \
  template void LayeredModel<T>::step_done(const BatchView &);                                                           \
  template int LayeredModel<T>::poll_errors();
ORION_INSTANTIATE(float)
ORION_INSTANTIATE(bf16)

}  // namespace orion
