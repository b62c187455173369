// What every device model shares: the streams and buffers of a step, the upload of weights and of the
// step's batch description, batch validation, the step graph, the LM head, replays and profiles. A model
// adds its weights and the kernel sequence of its layers (run_step_body). Mirrors the model-independent
// part of TransformerModel::forward (crates/orion-models/src/transformer.rs:359-442): the host only
// validates the batch, resolves slots (attention.rs:182-186) and launches.
#pragma once

#include <algorithm>
#include <cstdlib>
#include <cstring>
#include <map>
#include <tuple>
#include <vector>

#include "model.h"

namespace orion {

// Set from the environment (see model.cu).
extern bool g_step_graph;
extern const uint32_t kGraphAfterSteps;
constexpr size_t kMaxStepGraphs = 16;

template <typename T>
struct DTypeOf;
template <>
struct DTypeOf<float> { static constexpr int value = ORION_DTYPE_F32; static constexpr bool is_bf16 = false; };
template <>
struct DTypeOf<bf16> { static constexpr int value = ORION_DTYPE_BF16; static constexpr bool is_bf16 = true; };

inline size_t dtype_size(int dtype) {
  switch (dtype) {
    case ORION_DTYPE_F32: return 4;
    case ORION_DTYPE_F16:
    case ORION_DTYPE_BF16: return 2;
    default: return 0;
  }
}

// The sizes the shared code needs of a model.
struct StepShape {
  uint32_t hidden = 0, vocab = 0, max_positions = 0, num_blocks = 0, block_size = 0, max_batch_tokens = 0, max_batch_sequences = 0;
};

template <typename T>
class StepModel : public ModelBase {
 public:
  // Only the ordinal is kept: the model may outlive the backend handle it was created from.
  explicit StepModel(OrionBackend *backend) : ordinal_(backend->ordinal) {}
  ~StepModel() override {
    cudaSetDevice(ordinal_);
    if (stream_) cudaStreamSynchronize(stream_);
    drop_graphs();
    for (void *p : allocs_) cudaFree(p);
    if (h_meta_) cudaFreeHost(h_meta_);
    if (stage_raw_) cudaFree(stage_raw_);
    if (stage_f32_) cudaFree(stage_f32_);
    for (cudaEvent_t e : head_ev_)
      if (e) cudaEventDestroy(e);
    if (copy_stream_) cudaStreamDestroy(copy_stream_);
    if (ev0_) cudaEventDestroy(ev0_);
    if (ev1_) cudaEventDestroy(ev1_);
    for (cudaEvent_t e : prof_pool_) cudaEventDestroy(e);
    if (stream_) cudaStreamDestroy(stream_);
  }

  int forward(const BatchView &b, float *logits_out, uint64_t logits_capacity, uint32_t *token_ids_out) override;
  int replay(int iterations, uint32_t category_mask, float *elapsed_ms) override;
  int profile(int iterations, float category_ms[kProfCategories], uint64_t category_launches[kProfCategories]) override;
  uint64_t last_launch_count() const override { return last_launches_; }

 protected:
  // ---- what a model provides ----
  // part 0: the whole step; 1: the embedding and the layers (what a step graph holds); 2: the LM head and what follows
  virtual int run_step_body(bool want_argmax, int part) = 0;
  // Whether this step may be replayed as a graph, and the launch geometry that its layout alone does not fix.
  virtual bool graph_eligible() const = 0;
  virtual void graph_plan(uint32_t *splits, uint32_t *blocks_per_split) const = 0;
  // Model-specific batch checks (before anything is launched), after the shared ones.
  virtual int check_batch(const BatchView &) { return ORION_OK; }
  // Description of the batch's prompt portions for the prefill attention kernel; called for batches that are not
  // all single rows, before anything is launched. May use at most tile_words words at `t`.
  struct Meta;
  virtual size_t tile_words(uint64_t seqs, uint64_t rows) const { return 0; }
  virtual int fill_tiles(const BatchView &, uint32_t *t, Meta &) { return ORION_OK; }
  // Words of model-specific batch description; their number may depend on the sequence count only.
  virtual size_t extra_words(uint64_t) const { return 0; }
  virtual void fill_extra(const BatchView &, uint32_t *) {}
  virtual void step_done(const BatchView &) {}  // the step of a batch was launched and ended without an error
  virtual void step_failed() {}
  virtual float logit_softcap() const { return 0.f; }  // logits become cap * tanh(logit / cap); 0 = they stay
  virtual bool leader() const { return true; }  // only the leader of a group returns logits (Rank::is_leader)
  virtual bool out_rows_fixed() const { return false; }  // the output buffers cannot move (peers hold their address)
  // Device error words set by bounded waits that ran out.
  virtual int poll_errors() {
    uint32_t code = 0;
    if (!DTypeOf<T>::is_bf16) return ORION_OK;
    ORION_TRY(gemm_tc_poll_error(&code));
    if (code) return set_error(ORION_ERR_BACKEND, "backend cuda failed at gemm: a bounded pipeline wait ran out (code %u)", code);
    return ORION_OK;
  }
  // Waits for a stream of this model.
  virtual int wait_for(cudaStream_t s, const char *stage) {
    ORION_CUDA_CHECK(stage, cudaStreamSynchronize(s));
    return ORION_OK;
  }

  // ---- shared ----
  int init_step(const StepShape &shape);
  template <typename U>
  int alloc(U **p, size_t count) {
    void *raw = nullptr;
    ORION_CUDA_CHECK("allocate", cudaMalloc(&raw, (count ? count : 1) * sizeof(U)));
    allocs_.push_back(raw);
    *p = static_cast<U *>(raw);
    return ORION_OK;
  }
  int ensure_stage(void **buf, size_t *cap, size_t bytes) {
    if (*cap >= bytes) return ORION_OK;
    if (*buf) cudaFree(*buf);
    *buf = nullptr;
    *cap = 0;
    ORION_CUDA_CHECK("allocate staging", cudaMalloc(buf, bytes));
    *cap = bytes;
    return ORION_OK;
  }
  // Copies rows [r0,r1) x cols [c0,c1) of a host [R][C] tensor of `dtype` into a
  // contiguous device destination (`dst_t` of T or `dst_f`, whichever is non-null),
  // converting once at load like the reference's loader (loader.rs:74-96).
  int upload_slice(T *dst_t, float *dst_f, const void *src, int dtype, uint64_t C, uint64_t r0,
                   uint64_t r1, uint64_t c0, uint64_t c1);
  // Fills `n` elements with N(0, std) drawn on the device; the values depend on (seed, draw number) only.
  int fill_random(T *p, size_t n, uint64_t seed, float std) {
    ORION_TRY(ensure_stage(&stage_f32_, &stage_f32_cap_, std::min<size_t>(n, 64u << 20) * sizeof(float)));
    for (size_t off = 0; off < n; off += (64u << 20)) {
      const size_t m = std::min<size_t>(64u << 20, n - off);
      float *tmp = static_cast<float *>(stage_f32_);
      ORION_TRY(launch_fill_normal<float>(tmp, m, seed * 0x9E3779B97F4A7C15ull + (++random_draws_), stream_));
      ORION_TRY(launch_scale_convert<T>(tmp, p + off, m, std, stream_));  // N(0,1) -> N(0,std), narrowed to T
    }
    return ORION_OK;
  }
  int set_constant(float *p, size_t n, float value) {
    std::vector<float> v(n, value);
    ORION_CUDA_CHECK("init constant", cudaMemcpy(p, v.data(), n * sizeof(float), cudaMemcpyHostToDevice));
    return ORION_OK;
  }
  int run_step_graphed(bool want_argmax);
  int run_step(bool want_argmax) {
    const int rc = graph_eligible() ? run_step_graphed(want_argmax) : run_step_body(want_argmax, 0);
    if (rc != ORION_OK) step_failed();
    return rc;
  }
  // Room for `rows` rows of logits (and of the normalised rows they come from).
  int ensure_out_rows(uint64_t rows) {
    if (rows <= out_cap_) return ORION_OK;
    if (out_rows_fixed())
      return set_error(ORION_ERR_INVALID_REQUEST, "logits of %llu rows asked for, at most %llu under tensor parallelism",
                       (unsigned long long)rows, (unsigned long long)out_cap_);
    uint64_t cap = std::max<uint64_t>(out_cap_, 1);
    while (cap < rows) cap *= 2;
    ORION_TRY(alloc(&tail_, cap * shape_.hidden));
    ORION_TRY(alloc(&logits_, cap * shape_.vocab));
    ORION_TRY(alloc(&argmax_, cap));
    out_cap_ = cap;
    drop_graphs();  // captured steps write the previous buffers
    return ORION_OK;
  }
  // The projection plan for this many rows, cut back to what the partial buffer holds: it was sized at creation
  // under the tuning values of that moment, and a tuning call made since may ask for more k splits.
  GemmPlan plan_for(uint32_t rows, uint32_t n, uint32_t k, uint32_t ldx) const {
    GemmPlan p = gemm_plan(DTypeOf<T>::is_bf16, rows, n, k, ldx, k);
    while (p.splits > 1 && (size_t)p.splits * rows * n > partial_floats_) {
      --p.splits;
      if (!p.cluster_reduce) p.out_slabs = p.splits;
    }
    if (p.splits == 1) p.cluster_reduce = false, p.out_slabs = 1;
    return p;
  }
  int run_head(bool want_argmax);
  // Pure decode steps on one GPU replay a CUDA graph of the embedding and the layers once the same batch layout has
  // come 32 times in a row: every kernel argument of such a step is a pointer into buffers that do not move (the
  // step's tokens, positions and block tables are uploaded into the metadata array before the launch), so the graph
  // holds for as long as the layout (rows, sequences, offsets inside the metadata array, context splits) does.
  struct GraphKey {
    uint32_t rows, seqs, outs, splits, blocks_per_split, generation;
    size_t offsets[8];  // [7] is the address of the metadata array, the others are offsets inside it
    bool operator<(const GraphKey &o) const {
      return std::tie(rows, seqs, outs, splits, blocks_per_split, generation, offsets[0], offsets[1], offsets[2], offsets[3], offsets[4],
                      offsets[5], offsets[6], offsets[7]) <
             std::tie(o.rows, o.seqs, o.outs, o.splits, o.blocks_per_split, o.generation, o.offsets[0], o.offsets[1], o.offsets[2], o.offsets[3],
                      o.offsets[4], o.offsets[5], o.offsets[6], o.offsets[7]);
    }
    bool operator==(const GraphKey &o) const { return !(*this < o) && !(o < *this); }
  };
  struct StepGraph {
    cudaGraphExec_t exec = nullptr;
    uint64_t launches = 0;
  };
  std::map<GraphKey, StepGraph> graphs_;
  GraphKey last_key_{};
  uint32_t key_streak_ = 0;
  GraphKey layout_key() const {
    GraphKey key{};
    key.rows = meta_.rows, key.seqs = meta_.seqs, key.outs = meta_.outs, key.generation = g_tuning_generation;
    graph_plan(&key.splits, &key.blocks_per_split);
    // the tables (and the model-specific words) follow meta_.offsets at a distance that only depends on the sequence count
    const size_t offs[8] = {meta_.tokens, meta_.positions, meta_.slot_block, meta_.slot_slot, meta_.seq_of_row, meta_.last_rows,
                            meta_.offsets, reinterpret_cast<size_t>(d_meta_)};
    for (int i = 0; i < 8; ++i) key.offsets[i] = offs[i];
    return key;
  }
  void drop_graphs() {
    for (auto &g : graphs_)
      if (g.second.exec) cudaGraphExecDestroy(g.second.exec);
    graphs_.clear();
  }
  // Per-launch event pairs of a profiled step, resolved after the stream drains.
  struct ProfRec { int cat; cudaEvent_t a, b; };
  std::vector<ProfRec> prof_recs_;
  std::vector<cudaEvent_t> prof_pool_;
  size_t prof_used_ = 0;
  bool prof_on_ = false;
  uint32_t only_mask_ = 0;  // non-zero: launch only these kernel categories (timing replays)
  cudaEvent_t prof_event() {
    if (prof_used_ == prof_pool_.size()) {
      cudaEvent_t e = nullptr;
      cudaEventCreate(&e);
      prof_pool_.push_back(e);
    }
    return prof_pool_[prof_used_++];
  }
  template <typename F>
  int timed(int cat, F &&fn) {
    // Timing only: a replay restricted to some kernel categories launches just those, back to
    // back, on whatever the buffers hold (the results are meaningless, the shapes are the step's).
    if (only_mask_ && !(only_mask_ & (1u << cat))) return ORION_OK;
    if (!prof_on_) return fn();
    cudaEvent_t a = prof_event(), b = prof_event();
    cudaEventRecord(a, stream_);
    const int rc = fn();
    cudaEventRecord(b, stream_);
    prof_recs_.push_back({cat, a, b});
    return rc;
  }

  int ordinal_;
  StepShape shape_;
  cudaStream_t stream_ = nullptr;
  // LM head in column blocks with the download of block i overlapping the computation of i + 1
  static constexpr int kHeadChunks = 4;
  cudaStream_t copy_stream_ = nullptr;
  cudaEvent_t head_ev_[kHeadChunks] = {};
  uint32_t head_off_[kHeadChunks] = {}, head_cols_[kHeadChunks] = {};
  int head_chunks_ = 0;
  cudaEvent_t ev0_ = nullptr, ev1_ = nullptr;
  std::vector<void *> allocs_;
  T *embed_ = nullptr, *lm_head_ = nullptr;
  bool finalized_ = false;

  // work buffers
  float *hidden_ = nullptr, *partial_ = nullptr, *logits_ = nullptr;
  T *normed_ = nullptr, *tail_ = nullptr;
  uint32_t *argmax_ = nullptr;
  size_t partial_floats_ = 0;
  uint64_t out_cap_ = 0, random_draws_ = 0;

  // batch metadata: one u32 array on the device, filled from a pinned mirror
  uint32_t *d_meta_ = nullptr, *h_meta_ = nullptr;
  size_t meta_cap_ = 0;
  struct Meta {
    uint32_t rows = 0, seqs = 0, outs = 0, max_position = 0;
    uint64_t total_blocks = 0;  // sum over the rows of the blocks their contexts span
    bool decode = false, zero_count = false;
    size_t tokens = 0, positions = 0, slot_block = 0, slot_slot = 0, seq_of_row = 0, last_rows = 0,
           offsets = 0, extra = 0, tables = 0, tiles = 0, total = 0;
    uint32_t num_tiles = 0;  // prefill attention tiles (0 = the batch does not use that kernel)
    // Mixed batches: a run of one-token sequences at the head or the tail of the batch (the
    // scheduler puts all decodes before or after all prefills, scheduler.rs:244-250) goes to
    // the decode attention kernel, the other rows to the prefill kernel.
    uint32_t dec_row0 = 0, dec_rows = 0;
  } meta_;

  void *stage_raw_ = nullptr, *stage_f32_ = nullptr;
  size_t stage_raw_cap_ = 0, stage_f32_cap_ = 0;
  uint64_t last_launches_ = 0;
};

template <typename T>
int StepModel<T>::init_step(const StepShape &shape) {
  shape_ = shape;
  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  ORION_CUDA_CHECK("create stream", cudaStreamCreateWithFlags(&stream_, cudaStreamNonBlocking));
  ORION_CUDA_CHECK("create stream", cudaStreamCreateWithFlags(&copy_stream_, cudaStreamNonBlocking));
  for (cudaEvent_t &e : head_ev_) ORION_CUDA_CHECK("create event", cudaEventCreateWithFlags(&e, cudaEventDisableTiming));
  ORION_CUDA_CHECK("create event", cudaEventCreate(&ev0_));
  ORION_CUDA_CHECK("create event", cudaEventCreate(&ev1_));
  const size_t rows = shape.max_batch_tokens, H = shape.hidden;
  ORION_TRY(alloc(&hidden_, rows * H));
  ORION_TRY(alloc(&normed_, rows * H));
  return ensure_out_rows(shape.max_batch_sequences);
}

template <typename T>
int StepModel<T>::upload_slice(T *dst_t, float *dst_f, const void *src, int dtype, uint64_t C,
                           uint64_t r0, uint64_t r1, uint64_t c0, uint64_t c1) {
  const size_t es = dtype_size(dtype);
  const uint64_t rows = r1 - r0, cols = c1 - c0;
  if (rows == 0 || cols == 0) return ORION_OK;
  const bool direct = dst_t ? (dtype == DTypeOf<T>::value) : (dtype == ORION_DTYPE_F32);
  const size_t row_bytes = cols * es;
  uint64_t chunk_rows = std::max<uint64_t>(1, (64ull << 20) / std::max<size_t>(row_bytes, 1));
  for (uint64_t r = 0; r < rows; r += chunk_rows) {
    const uint64_t nr = std::min(chunk_rows, rows - r);
    const uint8_t *s = static_cast<const uint8_t *>(src) + ((r0 + r) * C + c0) * es;
    const size_t n = nr * cols;
    void *direct_dst = dst_t ? static_cast<void *>(dst_t + r * cols) : static_cast<void *>(dst_f + r * cols);
    if (direct) {
      ORION_CUDA_CHECK("upload tensor", cudaMemcpy2DAsync(direct_dst, row_bytes, s, C * es, row_bytes, nr,
                                                          cudaMemcpyHostToDevice, stream_));
      ORION_CUDA_CHECK("upload tensor", cudaStreamSynchronize(stream_));
      continue;
    }
    ORION_TRY(ensure_stage(&stage_raw_, &stage_raw_cap_, n * es));
    ORION_CUDA_CHECK("upload tensor", cudaMemcpy2DAsync(stage_raw_, row_bytes, s, C * es, row_bytes, nr,
                                                        cudaMemcpyHostToDevice, stream_));
    // widen to f32 unless the source already is
    const float *as_f32 = nullptr;
    if (dtype == ORION_DTYPE_F32) {
      as_f32 = static_cast<const float *>(stage_raw_);
    } else {
      float *wide = nullptr;
      if (dst_f) {
        wide = dst_f + r * cols;
      } else {
        ORION_TRY(ensure_stage(&stage_f32_, &stage_f32_cap_, n * sizeof(float)));
        wide = static_cast<float *>(stage_f32_);
      }
      if (dtype == ORION_DTYPE_BF16)
        ORION_TRY(launch_convert_to_f32<bf16>(static_cast<const bf16 *>(stage_raw_), wide, n, stream_));
      else
        ORION_TRY(launch_f16_to_f32(static_cast<const uint16_t *>(stage_raw_), wide, n, stream_));
      as_f32 = wide;
    }
    if (dst_t) ORION_TRY(launch_convert_from_f32<T>(as_f32, dst_t + r * cols, n, stream_));
    ORION_CUDA_CHECK("upload tensor", cudaStreamSynchronize(stream_));
  }
  return ORION_OK;
}

template <typename T>
int StepModel<T>::run_step_graphed(bool want_argmax) {
  const GraphKey key = layout_key();
  key_streak_ = (key_streak_ > 0 && key == last_key_) ? key_streak_ + 1 : 1;
  last_key_ = key;
  auto it = graphs_.find(key);
  if (it == graphs_.end() && key_streak_ >= kGraphAfterSteps) {
    if (graphs_.size() >= kMaxStepGraphs) drop_graphs();
    cudaGraph_t graph = nullptr;
    StepGraph sg;  // stays without an executable graph if anything below fails: the layout is then launched kernel by kernel
    const uint64_t before = g_launch_count;
    if (cudaStreamBeginCapture(stream_, cudaStreamCaptureModeThreadLocal) == cudaSuccess) {
      const int rc = run_step_body(false, 1);
      const cudaError_t ce = cudaStreamEndCapture(stream_, &graph);
      sg.launches = g_launch_count - before;
      if (rc != ORION_OK || ce != cudaSuccess || cudaGraphInstantiate(&sg.exec, graph, 0) != cudaSuccess) sg.exec = nullptr;
      if (graph) cudaGraphDestroy(graph);
    }
    g_launch_count = before;
    if (!sg.exec) {
      cudaGetLastError();  // the failed capture's error is not the step's
      clear_error();
    }
    it = graphs_.emplace(key, sg).first;
  }
  if (it != graphs_.end() && it->second.exec) {
    ORION_CUDA_CHECK("step graph launch", cudaGraphLaunch(it->second.exec, stream_));
    g_launch_count += it->second.launches;
  } else {
    ORION_TRY(run_step_body(want_argmax, 1));
  }
  return run_step_body(want_argmax, 2);
}


template <typename T>
int StepModel<T>::run_head(bool want_argmax) {
  constexpr bool kBf16 = DTypeOf<T>::is_bf16;
  const uint32_t S = meta_.outs, H = shape_.hidden, V = shape_.vocab;
  GemmPlan hp = gemm_plan(kBf16, S, V, H, H, H);
  hp.splits = hp.out_slabs = 1, hp.cluster_reduce = false;  // logits are written in place, row-major [S][V]
  head_chunks_ = 0;
  auto cap = [&](uint32_t n0, uint32_t n) -> int {
    const float c = logit_softcap();
    return c == 0.f ? ORION_OK : timed(kProfElementwise, [&] { return launch_softcap(logits_ + n0, S, n, V, c, stream_); });
  };
  if (kBf16 && hp.tensor_core && V >= 4 * 8192 && !want_argmax) {
    // A large vocabulary goes out in column blocks, an event after each: forward() copies block i
    // to the host (copy engine, second stream) while block i + 1 is being computed.
    const uint32_t per = (((V + 127) / 128 + kHeadChunks - 1) / kHeadChunks) * 128;
    for (uint32_t c = 0; c < (uint32_t)kHeadChunks && c * per < V; ++c) {
      const uint32_t n0 = c * per, nn = std::min(per, V - n0);
      GemmPlan cp = hp;
      cp.ldc = V;
      ORION_TRY(timed(kProfGemm, [&] { return launch_gemm<T>(tail_, H, lm_head_ + (size_t)n0 * H, H, logits_ + n0, S, nn, H, cp, stream_); }));
      ORION_TRY(cap(n0, nn));
      ORION_CUDA_CHECK("lm head", cudaEventRecord(head_ev_[c], stream_));
      head_off_[c] = n0;
      head_cols_[c] = nn;
      head_chunks_ = c + 1;
    }
    return ORION_OK;
  }
  ORION_TRY(timed(kProfGemm, [&] { return launch_gemm<T>(tail_, H, lm_head_, H, logits_, S, V, H, hp, stream_); }));
  ORION_TRY(cap(0, V));
  if (want_argmax) ORION_TRY(timed(kProfElementwise, [&] { return launch_argmax(logits_, S, V, argmax_, stream_); }));
  return ORION_OK;
}

template <typename T>
int StepModel<T>::forward(const BatchView &b, float *logits_out, uint64_t logits_capacity,
                      uint32_t *token_ids_out) {
  const StepShape &d = shape_;
  if (!finalized_) return set_error(ORION_ERR_MODEL, "model weights are not finalized");
  // ForwardBatch::validate (orion-core/src/traits.rs:232-261)
  const uint64_t S = b.num_sequences;
  if (b.num_slot_token_counts != S || b.num_context_lens != S || b.num_block_tables != S)
    return set_error(ORION_ERR_INTERNAL,
                     "ForwardBatch arrays disagree: %llu sequence ids, %llu token counts, %llu context "
                     "lens, %llu block tables",
                     (unsigned long long)S, (unsigned long long)b.num_slot_token_counts,
                     (unsigned long long)b.num_context_lens, (unsigned long long)b.num_block_tables);
  if (b.num_positions != b.num_tokens)
    return set_error(ORION_ERR_INTERNAL, "ForwardBatch has %llu tokens but %llu positions",
                     (unsigned long long)b.num_tokens, (unsigned long long)b.num_positions);
  // Malformed calls across the C boundary (the Rust vectors cannot be null or out of order).
  if ((b.num_tokens > 0 && (!b.tokens || !b.positions)) || (S > 0 && (!b.slot_token_counts || !b.block_table_offsets)))
    return set_error(ORION_ERR_INVALID_REQUEST, "null batch array");
  for (uint64_t s = 0; s < S; ++s)
    if (b.block_table_offsets[s + 1] < b.block_table_offsets[s])
      return set_error(ORION_ERR_INVALID_REQUEST, "block table offsets decrease at sequence %llu", (unsigned long long)s);
  if (S > 0 && b.block_table_offsets[S] > 0 && !b.block_tables_flat)
    return set_error(ORION_ERR_INVALID_REQUEST, "null batch array");
  uint64_t summed = 0;
  for (uint64_t s = 0; s < S; ++s) summed += b.slot_token_counts[s];
  if (summed != b.num_tokens)
    return set_error(ORION_ERR_INTERNAL,
                     "ForwardBatch slot token counts sum to %llu but there are %llu tokens",
                     (unsigned long long)summed, (unsigned long long)b.num_tokens);
  last_launches_ = 0;
  if (b.num_tokens == 0) return ORION_OK;  // transformer.rs:361-367: empty batch, empty output
  const uint64_t Tn = b.num_tokens;
  if (Tn > d.max_batch_tokens || S > d.max_batch_sequences)
    return set_error(ORION_ERR_INVALID_REQUEST,
                     "batch of %llu tokens / %llu sequences exceeds the configured capacity (%u / %u)",
                     (unsigned long long)Tn, (unsigned long long)S, d.max_batch_tokens,
                     d.max_batch_sequences);
  // Rows whose logits are asked for: the last row of every sequence, or the caller's list.
  const uint64_t R = b.logit_rows ? b.num_logit_rows : S;
  for (uint64_t i = 0; b.logit_rows && i < R; ++i)
    if (b.logit_rows[i] >= Tn)
      return set_error(ORION_ERR_INVALID_REQUEST, "logits of row %u asked for in a batch of %llu rows", b.logit_rows[i],
                       (unsigned long long)Tn);
  if (logits_out && logits_capacity < R * (uint64_t)d.vocab)
    return set_error(ORION_ERR_INVALID_REQUEST, "logits buffer holds %llu floats, %llu needed",
                     (unsigned long long)logits_capacity, (unsigned long long)(R * (uint64_t)d.vocab));

  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  ORION_TRY(ensure_out_rows(R));
  const uint64_t table_entries = S ? b.block_table_offsets[S] : 0;
  Meta mt;
  mt.rows = (uint32_t)Tn;
  mt.seqs = (uint32_t)S;
  mt.outs = (uint32_t)R;
  mt.tokens = 0;
  mt.positions = Tn;
  mt.slot_block = 2 * Tn;
  mt.slot_slot = 3 * Tn;
  mt.seq_of_row = 4 * Tn;
  mt.last_rows = 5 * Tn;
  mt.offsets = 5 * Tn + R;
  mt.extra = mt.offsets + S + 1;
  mt.tables = mt.extra + extra_words(S);
  mt.tiles = mt.tables + table_entries;
  mt.total = mt.tiles + tile_words(S, Tn);
  if (table_entries > UINT32_MAX) return set_error(ORION_ERR_INVALID_REQUEST, "block tables too large");
  if (mt.total > meta_cap_) {
    const size_t cap = mt.total * 2 + 1024;
    if (h_meta_) cudaFreeHost(h_meta_);
    h_meta_ = nullptr;
    meta_cap_ = 0;
    ORION_CUDA_CHECK("allocate batch mirror", cudaMallocHost(reinterpret_cast<void **>(&h_meta_), cap * sizeof(uint32_t)));
    ORION_TRY(alloc(&d_meta_, cap));  // the previous device array stays owned until destruction
    drop_graphs();                    // captured steps point into the previous array
    meta_cap_ = cap;
  }
  uint32_t *h = h_meta_;
  // seq_of_row and slot resolution BEFORE any compute or KV write (transformer.rs:371-387).
  {
    uint64_t row = 0;
    for (uint64_t s = 0; s < S; ++s) {
      for (uint64_t c = 0; c < b.slot_token_counts[s]; ++c) h[mt.seq_of_row + row++] = (uint32_t)s;
      if (b.slot_token_counts[s] == 0) mt.zero_count = true;
    }
  }
  const uint32_t B = d.block_size;
  bool all_single = true;
  for (uint64_t s = 0; s < S; ++s) all_single &= (b.slot_token_counts[s] == 1);
  for (uint64_t row = 0; row < Tn; ++row) {
    const uint32_t seq = h[mt.seq_of_row + row], pos = b.positions[row];
    const uint64_t t0 = b.block_table_offsets[seq], tlen = b.block_table_offsets[seq + 1] - t0;
    const uint64_t logical = pos / B;  // locate, attention.rs:182-186
    if (logical >= tlen)
      return set_error(ORION_ERR_INTERNAL, "position %u has no block in the table for sequence %u", pos, seq);
    h[mt.slot_block + row] = b.block_tables_flat[t0 + logical];
    h[mt.slot_slot + row] = pos % B;
    mt.max_position = std::max(mt.max_position, pos);
    mt.total_blocks += logical + 1;
  }
  for (uint64_t row = 0; row < Tn; ++row)  // embed, transformer.rs:211-217
    if (b.tokens[row] >= d.vocab)
      return set_error(ORION_ERR_INTERNAL, "token id %u is outside the vocabulary of %u", b.tokens[row],
                       d.vocab);
  for (uint64_t row = 0; row < Tn; ++row)  // RoPE range, transformer.rs:255-262
    if (b.positions[row] >= d.max_positions)
      return set_error(ORION_ERR_INTERNAL, "position %u exceeds the RoPE table (%u entries)", b.positions[row],
                       d.max_positions);
  // Every block a query row will read must exist in the arena (attention.rs:150-155);
  // checked here so that no kernel ever sees an out-of-range block id.
  for (uint64_t row = 0; row < Tn; ++row) {
    const uint32_t seq = h[mt.seq_of_row + row];
    const uint64_t t0 = b.block_table_offsets[seq];
    const uint64_t used = (uint64_t)b.positions[row] / B + 1;
    for (uint64_t e = 0; e < used; ++e)
      if (b.block_tables_flat[t0 + e] >= d.num_blocks)
        return set_error(ORION_ERR_INTERNAL, "block %u out of range (have %u)", b.block_tables_flat[t0 + e],
                         d.num_blocks);
  }
  ORION_TRY(check_batch(b));
  std::memcpy(h + mt.tokens, b.tokens, Tn * sizeof(uint32_t));
  std::memcpy(h + mt.positions, b.positions, Tn * sizeof(uint32_t));
  {
    uint64_t cursor = 0;
    for (uint64_t s = 0; s < S; ++s) {  // transformer.rs:410-420
      cursor += b.slot_token_counts[s];
      if (!b.logit_rows) h[mt.last_rows + s] = (uint32_t)(cursor ? cursor - 1 : 0);
      h[mt.offsets + s] = (uint32_t)b.block_table_offsets[s];
    }
    h[mt.offsets + S] = (uint32_t)table_entries;
    if (b.logit_rows && R) std::memcpy(h + mt.last_rows, b.logit_rows, R * sizeof(uint32_t));
  }
  if (table_entries) std::memcpy(h + mt.tables, b.block_tables_flat, table_entries * sizeof(uint32_t));
  fill_extra(b, h + mt.extra);
  mt.decode = all_single;
  if (!all_single) ORION_TRY(fill_tiles(b, h + mt.tiles, mt));
  meta_ = mt;

  g_launch_count = 0;
  ORION_CUDA_CHECK("upload batch", cudaMemcpyAsync(d_meta_, h, mt.total * sizeof(uint32_t), cudaMemcpyHostToDevice, stream_));
  ORION_TRY(run_step(token_ids_out != nullptr));
  last_launches_ = g_launch_count;
  if (mt.zero_count) {
    ORION_TRY(wait_for(stream_, "forward"));
    // transformer.rs:413-417: detected after the layers ran, so KV slots were written.
    return set_error(ORION_ERR_INTERNAL, "a scheduled sequence contributed zero tokens");
  }
  if (!leader()) {
    ORION_TRY(wait_for(stream_, "forward"));
  } else {
    if (logits_out && R > 0 && head_chunks_ > 0) {
      const size_t pitch = (size_t)d.vocab * sizeof(float);
      for (int c = 0; c < head_chunks_; ++c) {  // block c leaves while the blocks after it are computed
        ORION_CUDA_CHECK("download logits", cudaStreamWaitEvent(copy_stream_, head_ev_[c], 0));
        ORION_CUDA_CHECK("download logits", cudaMemcpy2DAsync(logits_out + head_off_[c], pitch, logits_ + head_off_[c], pitch,
                                                              (size_t)head_cols_[c] * sizeof(float), R, cudaMemcpyDeviceToHost,
                                                              copy_stream_));
      }
      ORION_TRY(wait_for(copy_stream_, "download logits"));
    } else if (logits_out && R > 0) {
      ORION_CUDA_CHECK("download logits", cudaMemcpyAsync(logits_out, logits_, R * (size_t)d.vocab * sizeof(float),
                                                          cudaMemcpyDeviceToHost, stream_));
    }
    if (token_ids_out && R > 0)
      ORION_CUDA_CHECK("download tokens", cudaMemcpyAsync(token_ids_out, argmax_, R * sizeof(uint32_t),
                                                          cudaMemcpyDeviceToHost, stream_));
    ORION_TRY(wait_for(stream_, "forward"));
  }
  ORION_TRY(poll_errors());
  step_done(b);
  return ORION_OK;
}

template <typename T>
int StepModel<T>::replay(int iterations, uint32_t category_mask, float *elapsed_ms) {
  if (meta_.rows == 0 || meta_.zero_count)
    return set_error(ORION_ERR_INVALID_REQUEST, "replay needs a preceding successful forward");
  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  ORION_CUDA_CHECK("replay", cudaStreamSynchronize(stream_));
  only_mask_ = category_mask & ((1u << kProfCategories) - 1);
  // a layout that will be replayed as a graph is brought there before the clock starts
  for (uint32_t i = 0; i <= kGraphAfterSteps && graph_eligible() && graphs_.find(layout_key()) == graphs_.end(); ++i) {
    const int rc = run_step(false);
    if (rc != ORION_OK) {
      only_mask_ = 0;
      return rc;
    }
  }
  ORION_CUDA_CHECK("replay", cudaEventRecord(ev0_, stream_));
  for (int i = 0; i < iterations; ++i) {
    g_launch_count = 0;
    const int rc = run_step(false);
    if (rc != ORION_OK) {
      only_mask_ = 0;
      return rc;
    }
    last_launches_ = g_launch_count;
  }
  only_mask_ = 0;
  ORION_CUDA_CHECK("replay", cudaEventRecord(ev1_, stream_));
  ORION_TRY(wait_for(stream_, "replay"));
  ORION_CUDA_CHECK("replay", cudaEventSynchronize(ev1_));
  float ms = 0.f;
  ORION_CUDA_CHECK("replay", cudaEventElapsedTime(&ms, ev0_, ev1_));
  if (elapsed_ms) *elapsed_ms = ms;
  return ORION_OK;
}

template <typename T>
int StepModel<T>::profile(int iterations, float category_ms[kProfCategories],
                      uint64_t category_launches[kProfCategories]) {
  if (meta_.rows == 0 || meta_.zero_count)
    return set_error(ORION_ERR_INVALID_REQUEST, "profile needs a preceding successful forward");
  ORION_CUDA_CHECK("set device", cudaSetDevice(ordinal_));
  for (int c = 0; c < kProfCategories; ++c) {
    category_ms[c] = 0.f;
    category_launches[c] = 0;
  }
  for (int i = 0; i < iterations; ++i) {
    prof_recs_.clear();
    prof_used_ = 0;
    prof_on_ = true;
    const int rc = run_step(false);
    prof_on_ = false;
    ORION_TRY(rc);
    ORION_CUDA_CHECK("profile", cudaStreamSynchronize(stream_));
    for (const ProfRec &r : prof_recs_) {
      float ms = 0.f;
      ORION_CUDA_CHECK("profile", cudaEventElapsedTime(&ms, r.a, r.b));
      category_ms[r.cat] += ms;
      category_launches[r.cat] += 1;
    }
  }
  return ORION_OK;
}

}  // namespace orion
