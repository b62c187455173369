// Layer-list models: the kernel sequence of a step (layered.h has the blocks).
#include "layered.h"

namespace orion {

template <typename T>
int LayeredModel<T>::mixer(const Layer &L, const T *x, SublayerOutput *y) {
  const uint32_t Tn = meta_.rows, H = d_.hidden_size;
  const GemmPlan p = plan_for(Tn, L.mix_in, H, H);
  const size_t slab = (size_t)Tn * L.mix_in;
  ORION_TRY(timed(kProfGemm, [&] { return launch_gemm<T>(x, H, L.w_mix, H, partial_, Tn, L.mix_in, H, p, stream_); }));
  if (L.gate_at && y) set_gate(p, L.mix_in, L.gate_at, L.gate_bias, y);
  if (L.latent()) return latent_attention(L, p, slab);
  if (L.attention()) return attention(L, p, slab);
  if (L.linear()) return linear_attention(L, p, slab);
  return timed(kProfAttention, [&] { return launch_min_gru<T>(partial_, p.out_slabs, slab, L.mix_bias, L.rec_state, state_batch(), cat_, L.cat, L.d.width, stream_); });
}

template <typename T>
int LayeredModel<T>::latent_attention(const Layer &L, const GemmPlan &p, size_t slab) {
  const uint32_t Tn = meta_.rows;
  const AttnBatch ab = attn_batch();
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

// Rows that decode read the cache by themselves, prompt portions in tiles; the rows' own keys and values are in the cache by then.
template <typename T>
int LayeredModel<T>::attention(const Layer &L, const GemmPlan &p, size_t slab) {
  const uint32_t Tn = meta_.rows;
  const AttnBatch ab = attn_batch();
  AttnForm form = L.form;
  form.gate = L.d.head_gate ? gate_ : nullptr;
  form.value_gate = L.d.value_gate ? value_gate_ : nullptr;
  ORION_TRY(timed(kProfElementwise, [&] {
    return launch_attention_prepare<T>(partial_, p.out_slabs, slab, L.in, ab.query_positions, d_meta_ + meta_.slot_block, d_meta_ + meta_.slot_slot,
                                       qbuf_, L.cache, L.kv, 0, L.d.head_gate ? gate_ : nullptr, Tn, stream_,
                                       L.d.value_gate ? value_gate_ : nullptr);
  }));
  if constexpr (DTypeOf<T>::is_bf16) {
    if (L.tuned) {
      if (few_rows_ > 0) {
        form.first_row = d_meta_ + meta_.extra, form.row_list = form.first_row + 3 * meta_.seqs + 1;
        const uint32_t sp = context_splits(L, few_rows_);
        const DecodeScratch sc = decode_scratch_at(scratch_, few_rows_, L.d.heads, L.d.kv_heads, L.kv.v_dim(), sp);
        ORION_TRY(timed(kProfAttention, [&] {
          return launch_paged_attention_decode_form(qbuf_, L.cache, L.kv, 0, ab, few_rows_, L.d.heads, sp, sc, form, cat_, stream_);
        }));
      }
      for (const TileSet &set : tile_sets_) {
        if (set.positions != 128 / (L.d.heads / L.d.kv_heads) || set.count == 0) continue;
        const auto *tiles = reinterpret_cast<const PrefillTile *>(d_meta_ + meta_.tiles + set.offset);
        ORION_TRY(timed(kProfAttention, [&] {
          return launch_paged_attention_prefill_form(qbuf_, L.cache, L.kv, 0, ab, tiles, set.count, L.d.heads, form, cat_, stream_);
        }));
      }
      return ORION_OK;
    }
  }
  return timed(kProfAttention, [&] { return launch_paged_attention_generic<T>(qbuf_, L.cache, L.kv, 0, ab, L.d.heads, cat_, stream_, form); });
}

// Sequences with few rows go token by token, longer portions in chunks.
template <typename T>
int LayeredModel<T>::linear_attention(const Layer &L, const GemmPlan &p, size_t slab) {
  const GlaWeights<T> w{L.w_decay, L.mix_bias, L.out_norm};
  uint32_t most = UINT32_MAX;
  if constexpr (DTypeOf<T>::is_bf16) {
    if (gla_chunks_supported(L.gla)) {
      most = kFewRows;
      if (gla_chunks_ > 0) {
        const uint32_t *lists = d_meta_ + meta_.tiles + gla_at_;
        const GlaPortions portions{reinterpret_cast<const GlaChunk *>(lists + 4 * meta_.seqs), reinterpret_cast<const GlaPortion *>(lists), gla_chunks_,
                                   gla_portions_};
        ORION_TRY(timed(kProfAttention, [&] {
          return launch_gla_chunks(partial_, p.out_slabs, slab, L.gla, w, L.rec_state, state_batch(), portions, gla_scratch_, cat_, L.cat, stream_);
        }));
      }
      if (few_rows_ == 0) return ORION_OK;
    }
  }
  return timed(kProfAttention, [&] {
    return launch_gla_steps<T>(partial_, p.out_slabs, slab, L.gla, w, L.rec_state, state_batch(), most, cat_, L.cat, stream_);
  });
}

template <typename T>
int LayeredModel<T>::dense_up(const Layer &L, const T *x, T *act, uint32_t ld) {
  const uint32_t Tn = meta_.rows, H = d_.hidden_size, F = L.d.ffn_dim;
  const bool relu2 = L.d.activation == ORION_ACT_RELU2;
  if (L.gated_ffn()) {
    const GemmPlan p = plan_for(Tn, 2 * F, H, H);
    if constexpr (DTypeOf<T>::is_bf16) {
      if (p.tensor_core && p.splits == 1)
        return timed(kProfGemm, [&] { return launch_gemm_act(x, H, L.w_up, H, act, ld, Tn, 2 * F, H, kGemmGeglu, stream_); });
    }
    ORION_TRY(timed(kProfGemm, [&] { return launch_gemm<T>(x, H, L.w_up, H, partial_, Tn, 2 * F, H, p, stream_); }));
    return timed(kProfElementwise, [&] {
      return launch_gated_act<T>(partial_, p.out_slabs, (size_t)Tn * 2 * F, GatedAct{kGatedGelu, 0.f}, act, ld, Tn, F, stream_);
    });
  }
  const GemmPlan p = plan_for(Tn, F, H, H);
  if constexpr (DTypeOf<T>::is_bf16) {
    if (p.tensor_core && p.splits == 1)  // the activation in the GEMM epilogue: no partials, no extra launch
      return timed(kProfGemm, [&] {
        return launch_gemm_act(x, H, L.w_up, H, act, ld, Tn, F, H, relu2 ? kGemmRelu2 : kGemmGelu, stream_, L.up_bias);
      });
  }
  ORION_TRY(timed(kProfGemm, [&] { return launch_gemm<T>(x, H, L.w_up, H, partial_, Tn, F, H, p, stream_); }));
  return timed(kProfElementwise, [&] {
    return launch_ffn_act<T>(partial_, p.out_slabs, (size_t)Tn * F, L.up_bias, relu2 ? kActRelu2 : kActGelu, act, ld, Tn, F, stream_);
  });
}

// The rows of x through their experts and the shared one; y names the results.
template <typename T>
int LayeredModel<T>::mixture(const Layer &L, const T *x, SublayerOutput *y) {
  const uint32_t Tn = meta_.rows, H = d_.hidden_size, E = L.moe.row_ld();
  float *shared_out = out_partial_ ? out_partial_ : partial_;
  const GemmPlan rp = plan_for(Tn, E, H, H);
  const MoePlan plan = moe_plan(DTypeOf<T>::is_bf16, L.moe, Tn);
  ORION_TRY(timed(kProfGemm, [&] { return launch_gemm<T>(x, H, L.w_router, H, partial_, Tn, E, H, rp, stream_); }));
  ORION_TRY(timed(kProfElementwise, [&] { return launch_moe_route<T>(partial_, rp.out_slabs, (size_t)Tn * E, L.correction, x, L.moe, plan, moe_, Tn, stream_); }));
  ORION_TRY(timed(kProfGemm, [&] {
    return launch_moe_experts<T>(x, L.e_up, L.e_down, L.s_up, L.s_down, L.moe, plan, moe_, shared_out, Tn, stream_);
  }));
  if (L.ff_gate_at) set_gate(rp, E, L.ff_gate_at, L.ff_gate_bias, y);
  if (L.moe.shared_ffn) y->partial = shared_out, y->splits = plan.down_splits, y->split_stride = (size_t)Tn * H;
  y->rows = moe_.down, y->place = moe_.place, y->top = L.moe.top;
  y->rows_splits = plan.down_splits, y->rows_stride = (size_t)Tn * L.moe.top * H;
  if (L.moe.weigh_output) y->weight = moe_.score;
  y->identity = x;
  return ORION_OK;
}

template <typename T>
int LayeredModel<T>::run_parallel_layers() {
  const uint32_t Tn = meta_.rows, H = d_.hidden_size, taps = d_.conv_taps;
  const uint32_t *m = d_meta_, *tokens = m + meta_.tokens;
  const float eps = (float)d_.norm_eps;
  const StateBatch sb = state_batch();
  // Decode batches take the residual add (or the embedding), the norm and the convolutions in one kernel.
  const bool fused = sb.single && residual_norm_conv_supported(H, taps);
  GemmPlan out{};
  for (uint32_t l = 0; l < d_.num_layers; ++l) {
    const Layer &L = layers_[l];
    T *ff_in = L.has_ffn() ? conv_f_ : nullptr;
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
    if (L.has_ffn()) ORION_TRY(dense_up(L, conv_f_, cat_ + L.ff_at, L.ff_ld));
    ORION_TRY(mixer(L, conv_m_));
    out = plan_for(Tn, H, L.cat, L.cat);
    ORION_TRY(timed(kProfGemm, [&] { return launch_gemm<T>(cat_, L.cat, L.w_out, L.cat, partial_, Tn, H, L.cat, out, stream_); }));
  }
  if (meta_.outs == 0) return ORION_OK;
  return timed(kProfElementwise, [&] {
    return launch_residual_rmsnorm<T>(partial_, out.out_slabs, (size_t)Tn * H, hidden_, final_norm_, eps, tail_, m + meta_.last_rows,
                                      meta_.outs, H, stream_);
  });
}

template <typename T>
int LayeredModel<T>::run_sandwich_layers() {
  const uint32_t Tn = meta_.rows, H = d_.hidden_size;
  const uint32_t *m = d_meta_;
  const float eps = (float)d_.norm_eps, mult = (float)d_.residual_mult;
  ORION_TRY(timed(kProfElementwise, [&] {
    return launch_embed_rmsnorm<T>(embed_, m + meta_.tokens, layers_[0].norm, eps, hidden_, normed_, Tn, H, stream_);
  }));
  // Adds a sublayer's output; `next` is the norm of what reads the sum, null at the end of the model.
  auto join = [&](const SublayerOutput &y, const float *post, const float *next) -> int {
    if (!next && meta_.outs == 0) return ORION_OK;
    return timed(kProfElementwise, [&] {
      return next ? launch_post_norm_residual<T>(y, hidden_, post, mult, next, eps, normed_, nullptr, Tn, H, stream_)
                  : launch_post_norm_residual<T>(y, hidden_, post, mult, final_norm_, eps, tail_, m + meta_.last_rows, meta_.outs, H, stream_);
    });
  };
  auto projected = [&](const T *x, const T *w, uint32_t k, const float *bias, SublayerOutput *y) -> int {
    const GemmPlan p = plan_for(Tn, H, k, k);
    y->partial = partial_, y->splits = p.out_slabs, y->split_stride = (size_t)Tn * H, y->bias = bias;
    return timed(kProfGemm, [&] { return launch_gemm<T>(x, k, w, k, partial_, Tn, H, k, p, stream_); });
  };
  for (uint32_t l = 0; l < d_.num_layers; ++l) {
    const Layer &L = layers_[l];
    const float *following = l + 1 < d_.num_layers ? layers_[l + 1].norm : nullptr;
    SublayerOutput y;
    ORION_TRY(mixer(L, normed_));
    ORION_TRY(projected(cat_, L.w_out, L.cat, nullptr, &y));
    ORION_TRY(join(y, L.norm_post, L.has_ffn() ? L.norm2 : following));
    if (!L.has_ffn()) continue;
    y = SublayerOutput{};
    if (L.moe.experts) {
      ORION_TRY(mixture(L, normed_, &y));
    } else {
      ORION_TRY(dense_up(L, normed_, cat_, L.ff_ld));
      ORION_TRY(projected(cat_, L.w_down, L.ff_ld, L.down_bias, &y));
    }
    ORION_TRY(join(y, L.norm2_post, following));
  }
  return ORION_OK;
}

template <typename T>
int LayeredModel<T>::run_prenorm_layers() {
  const uint32_t Tn = meta_.rows, H = d_.hidden_size;
  const uint32_t *m = d_meta_, *tokens = m + meta_.tokens;
  const float eps = (float)d_.norm_eps, mult = (float)d_.residual_mult, scale = (float)d_.embed_scale;
  ORION_TRY(timed(kProfElementwise, [&] {
    return launch_embed_rmsnorm<T>(embed_, tokens, layers_[0].norm, eps, hidden_, normed_, Tn, H, stream_, scale, layers_[0].shift);
  }));
  // Adds a sublayer's output, and ahead of the layer run `next` what belongs there; the sum is normalised for its reader.
  auto join = [&](const SublayerOutput &y, const float *norm, const Layer *next) -> int {
    StreamAddition<T> add;
    if (next) add = StreamAddition<T>{next->restart ? embed_ : nullptr, tokens, scale, next->shift};
    return timed(kProfElementwise, [&] { return launch_sublayer_residual<T>(y, hidden_, mult, add, norm, eps, normed_, nullptr, Tn, H, stream_); });
  };
  auto finish = [&](const SublayerOutput &y) -> int {
    if (meta_.outs == 0) return ORION_OK;
    return timed(kProfElementwise, [&] {
      return launch_sublayer_residual<T>(y, hidden_, mult, StreamAddition<T>{}, final_norm_, eps, tail_, m + meta_.last_rows, meta_.outs, H, stream_);
    });
  };
  auto projected = [&](const T *x, const T *w, uint32_t k, SublayerOutput *y) -> int {
    const GemmPlan p = plan_for(Tn, H, k, k);
    y->partial = partial_, y->splits = p.out_slabs, y->split_stride = (size_t)Tn * H;
    return timed(kProfGemm, [&] { return launch_gemm<T>(x, k, w, k, partial_, Tn, H, k, p, stream_); });
  };
  for (size_t l = 0; l < layers_.size(); ++l) {
    const Layer &L = layers_[l], *next = l + 1 < layers_.size() ? &layers_[l + 1] : nullptr;
    SublayerOutput y;
    ORION_TRY(mixer(L, normed_));
    ORION_TRY(projected(cat_, L.w_out, L.cat, &y));
    if (L.has_ffn()) {
      ORION_TRY(join(y, L.norm2, nullptr));
      y = SublayerOutput{};
      if (L.moe.experts) {
        ORION_TRY(mixture(L, normed_, &y));
      } else {
        ORION_TRY(dense_up(L, normed_, cat_, L.ff_ld));
        ORION_TRY(projected(cat_, L.w_down, L.ff_ld, &y));
      }
    }
    ORION_TRY(next ? join(y, next->norm, next) : finish(y));
  }
  return ORION_OK;
}

template <typename T>
int LayeredModel<T>::run_gated_postnorm_layers() {
  const uint32_t Tn = meta_.rows, H = d_.hidden_size;
  const uint32_t *m = d_meta_;
  const float eps = (float)d_.norm_eps, mult = (float)d_.residual_mult;
  ORION_TRY(timed(kProfElementwise, [&] {
    const EmbedTables<T> e{embed_, pairs_, places_, d_.bigram_buckets, d_.bigram_mul_prev, d_.bigram_mul_cur, history_, d_.block_size, (float)d_.embed_scale};
    const EmbedBatch b{m + meta_.tokens, m + meta_.positions, m + meta_.seq_of_row, m + meta_.slot_block, m + meta_.slot_slot, m + meta_.tables,
                       m + meta_.offsets, Tn};
    return launch_embed_tables<T>(e, b, hidden_, normed_, H, stream_);
  }));
  // Gates, normalises and adds a sublayer's output; what reads the sum next takes it as it is, at the end of the model normalised.
  auto join = [&](const SublayerOutput &y, const float *post, bool end) -> int {
    if (end && meta_.outs == 0) return ORION_OK;
    return timed(kProfElementwise, [&] {
      return end ? launch_gated_post_norm<T>(y, hidden_, post, mult, final_norm_, eps, tail_, m + meta_.last_rows, meta_.outs, H, stream_)
                 : launch_gated_post_norm<T>(y, hidden_, post, mult, nullptr, eps, normed_, nullptr, Tn, H, stream_);
    });
  };
  // partial_ holds the gate until the output has joined the stream
  auto projected = [&](const T *x, const T *w, uint32_t k, const float *bias, SublayerOutput *y) -> int {
    const GemmPlan p = plan_for(Tn, H, k, k);
    y->partial = out_partial_, y->splits = p.out_slabs, y->split_stride = (size_t)Tn * H, y->bias = bias;
    return timed(kProfGemm, [&] { return launch_gemm<T>(x, k, w, k, out_partial_, Tn, H, k, p, stream_); });
  };
  for (size_t l = 0; l < layers_.size(); ++l) {
    const Layer &L = layers_[l];
    const bool end = l + 1 == layers_.size();
    SublayerOutput y;
    ORION_TRY(mixer(L, normed_, &y));
    ORION_TRY(projected(cat_, L.w_out, L.cat, nullptr, &y));
    ORION_TRY(join(y, L.norm, end && !L.has_ffn()));
    if (!L.has_ffn()) continue;
    y = SublayerOutput{};
    if (L.moe.experts) {
      ORION_TRY(mixture(L, normed_, &y));
    } else {
      ORION_TRY(dense_up(L, normed_, cat_, L.ff_ld));
      const GemmPlan p = plan_for(Tn, H, H, H);
      ORION_TRY(timed(kProfGemm, [&] { return launch_gemm<T>(normed_, H, L.w_ff_gate, H, partial_, Tn, H, H, p, stream_); }));
      set_gate(p, H, 0, L.ff_gate_bias, &y);
      ORION_TRY(projected(cat_, L.w_down, L.ff_ld, L.down_bias, &y));
    }
    ORION_TRY(join(y, L.norm2, end));
  }
  return ORION_OK;
}

template <typename T>
int LayeredModel<T>::run_step_body(bool want_argmax, int part) {
  if (part != 2)
    ORION_TRY(parallel() ? run_parallel_layers()
                         : (sandwich() ? run_sandwich_layers() : (gated_postnorm() ? run_gated_postnorm_layers() : run_prenorm_layers())));
  if (part == 1 || meta_.outs == 0) return ORION_OK;
  return run_head(want_argmax);
}

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

#define ORION_INSTANTIATE(T) template int LayeredModel<T>::run_step_body(bool, int);
ORION_INSTANTIATE(float)
ORION_INSTANTIATE(bf16)

}  // namespace orion
