// Launchers of the device kernels. Every pointer is a device pointer; every
// launcher enqueues on `stream` and returns an OrionStatus. `T` is the storage
// type of weights, activations and the KV arena (float for the correctness
// build, bf16 for the performance build). GEMM results are always f32
// "partials": `splits` slabs of [rows][n] that the consuming kernel sums, which
// fuses the split-K reduction into the next elementwise step.
#pragma once

#include "common.cuh"

namespace orion {

// Shape of the paged KV arena of one rank:
// [layer][block][local kv head][k|v][slot][dim] (K and V rows may differ in size). Each (block, head) owns one
// contiguous chunk holding its K rows followed by its V rows, so a decode CTA
// fetches a 16-token block of one head with a single bulk copy.
// With `swizzle` set (16-bit storage, head_dim a multiple of 64) the 16-byte
// groups of every row are XOR-permuted by (slot & 7): the linear bulk copy then
// lands in shared memory in a layout ldmatrix reads without bank conflicts.
struct KvLayout {
  uint32_t num_layers, num_blocks, num_kv_heads, block_size, head_dim, swizzle;
  uint32_t value_dim = 0;  // size of a V row; 0 = head_dim
  // Not 0: the values are the keys before their norm, which is one factor per token and gains that the queries carry. A chunk
  // then holds one set of rows, for both, followed by the factor of every slot in f32 (factor_elems elements of storage each).
  uint32_t factor_elems = 0;
  __host__ __device__ uint32_t v_dim() const { return value_dim ? value_dim : head_dim; }
  __host__ __device__ size_t row_elems() const {
    return factor_elems ? (size_t(block_size) * head_dim + 7) / 8 * 8 : size_t(block_size) * (head_dim + v_dim());
  }
  __host__ __device__ size_t chunk_elems() const { return row_elems() + (size_t(block_size) * factor_elems + 7) / 8 * 8; }
  __host__ __device__ size_t layer_elems() const {
    return size_t(num_blocks) * num_kv_heads * chunk_elems();
  }
  // Start of the row holding (layer, block, head, k|v, slot).
  __host__ __device__ size_t row(uint32_t layer, uint32_t block, uint32_t head, uint32_t is_v,
                                 uint32_t slot) const {
    return layer * layer_elems() + (size_t(block) * num_kv_heads + head) * chunk_elems() +
           (is_v && !factor_elems ? size_t(block_size) * head_dim + size_t(slot) * v_dim() : size_t(slot) * head_dim);
  }
  // Start of the factor of (layer, block, head, slot).
  __host__ __device__ size_t factor(uint32_t layer, uint32_t block, uint32_t head, uint32_t slot) const {
    return layer * layer_elems() + (size_t(block) * num_kv_heads + head) * chunk_elems() + row_elems() + size_t(slot) * factor_elems;
  }
  // Position of logical dim `d` inside the row of `slot`.
  __host__ __device__ uint32_t col(uint32_t slot, uint32_t d) const {
    return swizzle ? ((((d >> 3) ^ (slot & 7u)) << 3) | (d & 7u)) : d;
  }
};

// hidden[r] = embed[tokens[r]] (f32); normed[r] = rms_norm(hidden[r]) * w.
// (transformer.rs:208-223 fused with tensor.rs:143-163)
template <typename T>
int launch_embed_rmsnorm(const T *embed, const uint32_t *tokens, const float *norm_w, float eps,
                         float *hidden, T *normed, uint32_t rows, uint32_t hidden_size,
                         cudaStream_t stream, float scale = 1.f, const float *shift = nullptr);  // hidden = scale * embed (+ shift, one vector)

// An embedding made of several tables, and its rows in the storage type (not normalised): hidden[r] = scale * embed[token] +
// pairs[row] + places[position], out[r] = hidden[r]. The row of `pairs` (null: none) is (previous token * mul_prev + token *
// mul_cur) mod buckets, or `buckets` for a sequence's first token. A token whose predecessor came in an earlier step finds it in
// `history`, the token of every cache slot ([blocks][block_size], written here). places (null: none) holds a row per position.
template <typename T>
struct EmbedTables {
  const T *embed = nullptr, *pairs = nullptr, *places = nullptr;
  uint64_t buckets = 0, mul_prev = 0, mul_cur = 0;
  uint32_t *history = nullptr;
  uint32_t block_size = 0;
  float scale = 1.f;
};
struct EmbedBatch {
  const uint32_t *tokens, *positions, *seq_of_row, *slot_block, *slot_slot, *tables_flat, *table_offsets;
  uint32_t rows;
};
template <typename T>
int launch_embed_tables(EmbedTables<T> e, EmbedBatch b, float *hidden, T *out, uint32_t hidden_size, cudaStream_t stream);

// hidden[r] += sum_s partial[s][r] (+ nothing else); out[i] = rms_norm(hidden[src(i)]) * w,
// src(i) = row_map ? row_map[i] : i. With row_map the residual is not written
// back (used for the final norm over the last row of each sequence).
// (transformer.rs:330-336, 343-345, 401-428)
template <typename T>
int launch_residual_rmsnorm(const float *partial, uint32_t splits, size_t split_stride,
                            float *hidden, const float *norm_w, float eps, T *out,
                            const uint32_t *row_map, uint32_t out_rows, uint32_t hidden_size,
                            cudaStream_t stream, uint32_t *ready = nullptr);  // ready: every CTA (one per output row) adds 1 when done

// Plain rms_norm of f32 rows into T (tensor.rs:143-163) for the op-level API.
template <typename T>
int launch_rmsnorm_rows(const float *x, const float *norm_w, float eps, T *out, uint32_t rows,
                        uint32_t cols, cudaStream_t stream);

// Sums the QKV partials (+bias), applies RoPE to q and k heads by table lookup
// at positions[r], writes q to `q_out` [rows][q_heads*hd] and k, v into the
// arena at (slot_block[r], slot_slot[r]). (transformer.rs:248-297, tensor.rs:283-298)
template <typename T>
int launch_rope_kvwrite(const float *partial, uint32_t splits, size_t split_stride,
                        const float *bias, const uint32_t *positions, const uint32_t *slot_block,
                        const uint32_t *slot_slot, const float *rope_cos, const float *rope_sin,
                        T *q_out, T *arena, KvLayout kv, uint32_t layer, uint32_t rows,
                        uint32_t q_heads, cudaStream_t stream);

// In-place RoPE over [rows][heads][hd] of T (op-level API; tensor.rs:283-298).
template <typename T>
int launch_rope_rows(T *x, const uint32_t *positions, const float *rope_cos, const float *rope_sin,
                     uint32_t rows, uint32_t heads, uint32_t head_dim, cudaStream_t stream);

// act[r][f] = silu(g) * u with g = sum_s partial[s][r][f], u = sum_s partial[s][r][ffn + f];
// `interleaved`: gate f and up f sit in columns 2f and 2f + 1 instead. (tensor.rs:167-189)
template <typename T>
int launch_swiglu(const float *partial, uint32_t splits, size_t split_stride, T *act, uint32_t rows,
                  uint32_t ffn, cudaStream_t stream, bool interleaved = false);
// The interleaved form with any gated activation and row stride `ldo`.
template <typename T>
int launch_gated_act(const float *partial, uint32_t splits, size_t split_stride, GatedAct f, T *act, uint32_t ldo, uint32_t rows, uint32_t ffn,
                     cudaStream_t stream);
// dst[r * dst_stride + c] = src[r * cols + c]
template <typename T>
int launch_copy_rows_strided(const T *src, T *dst, size_t rows, size_t cols, size_t dst_stride, cudaStream_t stream);

// out[r * ldo + c] = f(sum_s partial[s][r][c] + bias[c]), f = GELU (tanh form) or the square of relu; bias may be null.
enum FfnAct : uint32_t { kActGelu = 0, kActRelu2 = 1 };
template <typename T>
int launch_ffn_act(const float *partial, uint32_t splits, size_t split_stride, const float *bias, FfnAct f, T *out, uint32_t ldo, uint32_t rows,
                   uint32_t cols, cudaStream_t stream);

// A sublayer's output y that is normalised before it is added: hidden += mult * rms_norm(y) * post_w, then
// out[i] = rms_norm(hidden[src(i)]) * pre_w with src and row_map as in launch_residual_rmsnorm. y is the sum of a projection's
// slabs (partial may be null), a bias (may be null) and, where a row went through `top` experts, the rows place[r * top + k]
// of the experts' output (each the sum of rows_splits slabs).
struct SublayerOutput {
  const float *partial = nullptr;
  uint32_t splits = 0;
  size_t split_stride = 0;
  const float *bias = nullptr;
  const float *rows = nullptr;
  const uint32_t *place = nullptr;
  uint32_t top = 0, rows_splits = 0;
  size_t rows_stride = 0;
  const float *weight = nullptr;   // [rows][top] factors of the experts' rows; null = 1
  const void *identity = nullptr;  // [row][hidden] of T: what a choice with the place kNoPlace contributes
  // A gate per value, sigmoid(gate + gate_bias), from columns of a projection's slabs (row stride gate_ld). Null: none.
  const float *gate = nullptr, *gate_bias = nullptr;
  uint32_t gate_splits = 0, gate_ld = 0;
  size_t gate_stride = 0;
};
constexpr uint32_t kNoPlace = 0xFFFFFFFFu;
template <typename T>
int launch_post_norm_residual(SublayerOutput y, float *hidden, const float *post_w, float mult, const float *pre_w, float eps, T *out,
                              const uint32_t *row_map, uint32_t out_rows, uint32_t hidden_size, cudaStream_t stream);
// Pre-norm layers: the output joins as it is, hidden += mult * y, and what comes ahead of the next layer follows it:
// hidden += scale * embed[tokens[r]] (embed may be null), hidden += shift (a vector, may be null). `y.identity` may be `out`.
template <typename T>
struct StreamAddition {
  const T *embed = nullptr;
  const uint32_t *tokens = nullptr;
  float scale = 1.f;
  const float *shift = nullptr;
};
template <typename T>
int launch_sublayer_residual(SublayerOutput y, float *hidden, float mult, StreamAddition<T> add, const float *pre_w, float eps, T *out,
                             const uint32_t *row_map, uint32_t out_rows, uint32_t hidden_size, cudaStream_t stream);
// Post-norm layers: hidden += mult * rms_norm(gated y) * post_w, where the experts' weights and the gate count; out = rms_norm(hidden) *
// pre_w, or the rows of hidden themselves if pre_w is null.
template <typename T>
int launch_gated_post_norm(SublayerOutput y, float *hidden, const float *post_w, float mult, const float *pre_w, float eps, T *out,
                           const uint32_t *row_map, uint32_t out_rows, uint32_t hidden_size, cudaStream_t stream);
// x[r * ld + c] = cap * tanh(x[r * ld + c] / cap)
int launch_softcap(float *x, uint32_t rows, uint32_t cols, uint32_t ld, float cap, cudaStream_t stream);

// out[r][n] = sum_s partial[s][r][n] + bias[n]  (finishes tensor::linear, tensor.rs:126).
int launch_finish_linear(const float *partial, uint32_t splits, size_t split_stride,
                         const float *bias, float *out, uint32_t rows, uint32_t n,
                         cudaStream_t stream);

// First index of the strict row maximum; UINT32_MAX when nothing exceeds -inf.
// (orion-runtime/src/sampling.rs:196-206)
int launch_argmax(const float *logits, uint32_t rows, uint32_t cols, uint32_t *out,
                  cudaStream_t stream);

// Converts between f32 and T on the device (weight upload, arena read-back).
template <typename T>
int launch_convert_from_f32(const float *src, T *dst, size_t n, cudaStream_t stream);
template <typename T>
int launch_convert_to_f32(const T *src, float *dst, size_t n, cudaStream_t stream);
int launch_f16_to_f32(const uint16_t *src, float *dst, size_t n, cudaStream_t stream);
// dst[i][:] = src[row_map[i]][:]
template <typename T>
int launch_gather_rows(const T *src, const uint32_t *row_map, T *dst, uint32_t rows, uint32_t cols,
                       cudaStream_t stream);
// dst[i] = T(src[i] * scale)
template <typename T>
int launch_scale_convert(const float *src, T *dst, size_t n, float scale, cudaStream_t stream);

// Arena -> the reference's logical order [layer][block][k|v][slot][head][dim], f32.
template <typename T>
int launch_arena_to_reference_order(const T *arena, KvLayout kv, float *out, cudaStream_t stream);
// The reverse, for one layer given in reference order (op-level attention API).
template <typename T>
int launch_arena_from_reference_order(const float *ref, KvLayout kv, T *arena, cudaStream_t stream);

// Fills `n` elements with N(0, 1) values from a counter-based generator.
template <typename T>
int launch_fill_normal(T *dst, size_t n, uint64_t seed, cudaStream_t stream);

// ---- attention ---------------------------------------------------------------

struct AttnBatch {
  const uint32_t *query_positions;  // [rows] absolute position of each query row
  const uint32_t *seq_of_row;       // [rows]
  const uint32_t *tables_flat;      // concatenated block tables
  const uint32_t *table_offsets;    // [sequences + 1]
  uint32_t rows;
  uint32_t max_position;            // largest query position in the batch
};

// Which of the positions up to its own a query sees: the last `window` of them (0 = no window), of those the ones in
// its own chunk of `chunk` positions, counted from the sequence's start (0 = no chunks), and besides them the first `keep`
// positions of the sequence.
struct KeyRange {
  uint32_t window = 0, chunk = 0, keep = 0;
  // The first position of the run that ends with the query itself.
  __host__ __device__ uint32_t first(uint32_t pos) const {
    const uint32_t w = window && pos + 1 > window ? pos + 1 - window : 0, c = chunk ? pos / chunk * chunk : 0;
    return w > c ? w : c;
  }
  // Positions before that run which the query sees as well: 0 .. kept(pos) - 1.
  __host__ __device__ uint32_t kept(uint32_t pos) const {
    const uint32_t f = first(pos);
    return keep < f ? keep : f;
  }
  // Blocks of `size` positions before the one that the run begins in (`block0`) which hold kept positions.
  __host__ __device__ uint32_t kept_blocks(uint32_t block0, uint32_t size) const {
    const uint32_t n = (keep + size - 1) / size;
    return n < block0 ? n : block0;
  }
  // The most positions a query up to `max_position` sees.
  __host__ __device__ uint32_t most(uint32_t max_position) const {
    uint32_t n = max_position + 1;
    if (window && window < n && keep < n - window) n = window + keep;
    return chunk && chunk < n && keep < n - chunk ? chunk + keep : n;
  }
};
// What a design adds to causal attention over everything before; the defaults add nothing.
struct AttnForm {
  float scale = 0.f;              // of the scores; 0 = 1 / sqrt(head_dim)
  KeyRange range;
  const float *sinks = nullptr;   // [q_heads] logits that enter the denominator once and carry no value
  const float *gate = nullptr;    // [rows][q_heads] factors of the heads' outputs
  const void *value_gate = nullptr;  // [rows][q_heads * out_dim] of T: factors of the values
  float softcap = 0.f;            // scores become softcap * tanh(score / softcap); 0 = they stay
  // [q_heads]: dist_mult * ln(1 + dist_rate * (distance to the key)) is taken off every score. Null: nothing. The tuned kernels
  // take it where keys and values are one (KvLayout::factor_elems).
  const float *dist_mult = nullptr, *dist_rate = nullptr;
  uint32_t out_dim = 0, ldo = 0;  // values stored per head and row stride of the output; 0 = v_dim() and q_heads * out_dim
  // Decode only: the batch rows that decode (item i of the scratch belongs to row_list[i]), and the first row of every
  // sequence, since several rows of one sequence may decode together. Null: every row, one per sequence.
  const uint32_t *row_list = nullptr, *first_row = nullptr;
};

// Any shape, any mix of prefill and decode rows: one CTA per (row, query head),
// causal by absolute position (attention.rs:219-295).
template <typename T>
int launch_paged_attention_generic(const T *q, const T *arena, KvLayout kv, uint32_t layer,
                                   AttnBatch batch, uint32_t q_heads, T *out, cudaStream_t stream, AttnForm form = {});

// Folds the partial sums of a joint projection [q | k | v | g] (row stride `ld`): RMS norms over all heads of q and of k
// together (gains may be null: no norm), rotation of the first rope_dims dimensions of every head in neighbouring pairs
// (2i, 2i + 1) by the table's angles, q to `q_out` [rows][q_heads][kv.head_dim], k and v to the arena, and sigmoid(g), one
// value per query head, to `gate` [rows][q_heads] (may be null: no such columns). dim and value_dim are what the projection
// holds per head; the arena's rows may be longer, and what is beyond stays as it is.
//
// per_head: the other family of layouts. Every head is normalised by itself (gains of dim values, shared by the heads), dimension
// i rotates with i + rope_dims / 2 if `halves` is set, q, k and v have biases ([q | k | v], may be null), and g has a column per
// value: sigmoid(g) goes to `value_gate` [rows][q_heads * value_dim] (null: no such columns) instead of `gate`.
//
// keys_as_values (norms over all heads, nothing rotates, no gates): the projection holds [q | k] with biases ([q | k]). The cache gets
// k as projected and the factor of its norm (KvLayout::factor_elems); q_norm holds, per value of the queries, the queries' gain times
// that of the keys. The queries are also multiplied by q_factor[position] (null: 1).
struct AttnInputs {
  uint32_t q_heads, kv_heads, dim, value_dim, rope_dims, ld;
  float eps;
  const float *q_norm, *k_norm, *rope_cos, *rope_sin;
  bool per_head = false, halves = false;
  const float *bias = nullptr;
  bool keys_as_values = false;
  const float *q_factor = nullptr;
};
template <typename T>
int launch_attention_prepare(const float *partial, uint32_t splits, size_t split_stride, AttnInputs in, const uint32_t *positions,
                             const uint32_t *slot_block, const uint32_t *slot_slot, T *q_out, T *arena, KvLayout kv, uint32_t layer,
                             float *gate, uint32_t rows, cudaStream_t stream, T *value_gate = nullptr);
// K and V rows of one layer's arena as f32, [k|v][block][kv head][slot][dim] with dim values of a K row, value_dim of a V row.
template <typename T>
int launch_arena_rows(const T *arena, KvLayout kv, uint32_t dim, uint32_t value_dim, float *out, cudaStream_t stream);
// One value for all factors of an arena (KvLayout::factor_elems).
template <typename T>
int launch_fill_factors(T *arena, KvLayout kv, float value, cudaStream_t stream);

// Tuned prefill / mixed-batch path (bf16, head_dim 128, block 16): the batch is cut into
// tiles of consecutive rows of one sequence (prefill_tile_positions rows at most); one CTA per
// (kv head, tile) streams the sequence's K/V once for all rows of the tile.
struct PrefillTile {
  uint32_t row_start;     // first batch row of the tile
  uint32_t num_rows;      // rows (query positions) in the tile
  uint32_t seq;           // sequence the rows belong to
  uint32_t max_position;  // largest query position in the tile
};
bool prefill_attention_supported(KvLayout kv, uint32_t q_heads);
uint32_t prefill_tile_positions(uint32_t q_heads, uint32_t kv_heads);
int launch_paged_attention_prefill(const bf16 *q, const bf16 *arena, KvLayout kv, uint32_t layer,
                                   AttnBatch batch, const PrefillTile *tiles, uint32_t num_tiles,
                                   uint32_t q_heads, bf16 *out, cudaStream_t stream);
int prefill_poll_error(uint32_t *code);
// The same computation on tcgen05 / tensor memory (S and O accumulators in tensor memory, K/V tiles by
// tiled TMA straight out of the arena); same tiles, same arguments.
bool prefill_attention_tc_supported(KvLayout kv, uint32_t q_heads, const void *arena);
int launch_paged_attention_prefill_tc(const bf16 *q, const bf16 *arena, KvLayout kv, uint32_t layer,
                                      AttnBatch batch, const PrefillTile *tiles, uint32_t num_tiles,
                                      uint32_t q_heads, bf16 *out, cudaStream_t stream);
int prefill_tc_poll_error(uint32_t *code);
// Other forms of attention on the same kernels: head and value sizes of 64, 128 or 256 (an arena pads to them; above 128
// both 256), 16-token blocks. Their prefill tiles are 128 / (query heads per kv head) positions.
bool attention_form_supported(KvLayout kv, uint32_t q_heads);
// The size a head dimension is padded to in such an arena; 0 = no padding makes the kernels cover it.
inline uint32_t attention_padded_dim(uint32_t dim, uint32_t other) {
  if (dim == 0 || other == 0 || dim > 256 || other > 256) return 0;
  return dim > 128 || other > 128 ? 256 : (dim > 64 ? 128 : 64);
}
int launch_paged_attention_prefill_form(const bf16 *q, const bf16 *arena, KvLayout kv, uint32_t layer, AttnBatch batch,
                                        const PrefillTile *tiles, uint32_t num_tiles, uint32_t q_heads, AttnForm form, bf16 *out,
                                        cudaStream_t stream);

// Tuned decode path (bf16, head_dim 128, block 16, one query row per sequence):
// one CTA per (sequence, kv head, context split); the query heads of a GQA group
// share every K/V tile. `scratch` holds the per-split partial outputs.
struct DecodeScratch {
  float *partial_out;  // [rows][q_heads][max_splits][head_dim]
  float *partial_ml;   // [rows][q_heads][max_splits][2]  (running max, running sum)
  uint32_t max_splits;
  // [rows * kv_heads] arrival counters, zero between launches: the last CTA of a (row, kv head) to
  // finish merges the splits itself, so no separate combine launch follows. Null = combine kernel.
  uint32_t *counters;
  // 0: every row is cut into max_splits pieces; else a row of n blocks is cut into
  // round(n / blocks_per_split) pieces (at least 1, at most max_splits).
  uint32_t blocks_per_split;
};
// A scratch buffer starts with kDecodeCounterWords counter words (which must be zero when the buffer
// is first used and are left zero by every launch), followed by the partial results.
constexpr uint32_t kDecodeCounterWords = 16384;
bool decode_attention_supported(KvLayout kv, uint32_t q_heads);
// Floats a scratch buffer needs, counter words included.
size_t decode_scratch_floats(uint32_t rows, uint32_t q_heads, uint32_t head_dim,
                             uint32_t max_splits);
// Lays the parts of a scratch buffer of at least decode_scratch_floats(...) floats out.
DecodeScratch decode_scratch_at(float *base, uint32_t rows, uint32_t q_heads, uint32_t kv_heads, uint32_t head_dim,
                                uint32_t splits, uint32_t blocks_per_split = 0);
// Length-proportional context split for a ragged batch: `splits` = pieces of the longest row (the
// grid's z extent), `blocks_per_split` = blocks a piece should hold. `total_blocks` = sum over the
// rows of their block counts. splits == 1 means no row is cut.
struct DecodePlan {
  uint32_t splits, blocks_per_split;
};
DecodePlan decode_plan(uint32_t rows, uint32_t kv_heads, uint64_t total_blocks, uint32_t max_position,
                       uint32_t block_size, uint32_t max_splits);
uint32_t decode_choose_splits(uint32_t rows, uint32_t kv_heads, uint32_t max_position,
                              uint32_t block_size, uint32_t max_splits);
// With `partial` set the kernel takes the row's q, k and v straight from the QKV projection's
// f32 partial sums: it folds the split-K slabs, adds the bias, applies RoPE at the row's position
// (transformer.rs:248-297), writes k and v into the arena slot and uses them for this step, so no
// separate RoPE / KV-write kernel runs and `q` is not read.
struct FusedQkv {
  const float *partial = nullptr;  // [slabs][rows][(q_heads + 2 kv_heads) * head_dim]
  uint32_t slabs = 0;
  size_t slab_stride = 0;
  const float *bias = nullptr;     // [(q_heads + 2 kv_heads) * head_dim] or null
  const float *rope_cos = nullptr, *rope_sin = nullptr;  // [max_pos][head_dim / 2]
  const uint32_t *slot_block = nullptr;                  // [rows] physical block of the row's position
  bf16 *arena = nullptr;           // writable view of the arena
};
int launch_paged_attention_decode(const bf16 *q, const bf16 *arena, KvLayout kv, uint32_t layer,
                                  AttnBatch batch, uint32_t q_heads, uint32_t splits,
                                  DecodeScratch scratch, bf16 *out, cudaStream_t stream,
                                  FusedQkv fused = {});
// The same for other forms of attention and any number of query heads per kv head (eight share a CTA); `rows` of the
// batch are those of form.row_list.
uint32_t decode_form_splits(KvLayout kv, uint32_t q_heads, uint32_t rows, uint32_t most_keys);
int launch_paged_attention_decode_form(const bf16 *q, const bf16 *arena, KvLayout kv, uint32_t layer, AttnBatch batch, uint32_t rows,
                                       uint32_t q_heads, uint32_t splits, DecodeScratch scratch, AttnForm form, bf16 *out,
                                       cudaStream_t stream);
// Tuning: ring depth per warp (2..4) and the CTA count the context split aims for (0 keeps it).
void decode_set_tuning(int stages, uint32_t cta_target);
// Device error word of the decode kernel (0 = none); reading clears it.
int decode_poll_error(uint32_t *code);

// ---- state carried from token to token -----------------------------------------------
//
// Models with recurrent layers keep, besides the paged cache, a fixed amount of state per sequence. A
// state buffer holds two copies of every slot: a step reads the copy `read` of each of its sequences
// and writes the copy `write`, so no thread can meet a value of this step where it expects the previous
// one, and a step that is run again (a replay, a retry after an error) finds its inputs unchanged.
struct StateBatch {
  const uint32_t *first_row;  // [sequences + 1] batch rows of each sequence: [first_row[s], first_row[s + 1])
  const uint32_t *read;       // [sequences] copy to read; kNoState: the sequence starts here, all zeros
  const uint32_t *write;      // [sequences] copy to write
  const uint32_t *seq_of_row; // [rows]
  uint32_t rows, seqs;
  bool single;                // every sequence has exactly one row
};
constexpr uint32_t kNoState = 0xFFFFFFFFu;

// Causal per-channel convolution over time added to its input, for up to two sets of weights at once
// (the two sublayers of a parallel layer): out_i = h + conv_i(h), conv_i(h)_t = sum_j w_i[c][j] h_(t - taps + 1 + j).
// The filters are stored by tap, w_i[j][c]. `state` is [copies][taps - 1][cols]: the last taps - 1 rows of h. w2 / out2
// may be null.
template <typename T>
int launch_causal_conv(const T *h, const T *w1, const T *w2, uint32_t taps, T *state, StateBatch sb, T *out1, T *out2,
                       uint32_t cols, cudaStream_t stream);
// One row per sequence: residual add (as launch_residual_rmsnorm) or, with `tokens`, the embedding lookup,
// then the norm and the convolutions, in one kernel.
template <typename T>
int launch_residual_norm_conv(const float *partial, uint32_t splits, size_t split_stride, const T *embed, const uint32_t *tokens,
                              float *hidden, const float *norm_w, float eps, const T *w1, const T *w2, uint32_t taps, T *state,
                              StateBatch sb, T *out1, T *out2, uint32_t cols, cudaStream_t stream);
// dst[c][r] = src[r][c]
template <typename T>
int launch_transpose(const T *src, T *dst, uint32_t rows, uint32_t cols, cudaStream_t stream);
bool residual_norm_conv_supported(uint32_t cols, uint32_t taps);

// Minimal gated recurrence, element by element: with the projections' partial sums [z | x | g] of `width`
// columns each, z' = sigmoid(z + bias_z), u = x + bias_x, c = u >= 0 ? u + 1/2 : sigmoid(u),
// S_t = (1 - z') S_(t-1) + z' c, out = S_t * silu(g). `state` is [copies][width] in f32.
template <typename T>
int launch_min_gru(const float *partial, uint32_t splits, size_t split_stride, const float *bias, float *state, StateBatch sb,
                   T *out, uint32_t ldo, uint32_t width, cudaStream_t stream);

// Gated linear attention: per head a state S of dim x value_dim, S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t,
// out = rms_norm(o_t) * norm * silu(g). The joint projection holds [q | k | v | g | a] per row (row stride ld), a of `rank` values for
// all heads; q is scaled by dim^(-1/2), alpha = sigmoid(W a + bias)^(1 / tau), one value per key channel, W [heads * dim][rank].
// `state` is [copies][heads][dim][value_dim] in f32.
struct GlaShape {
  uint32_t heads, dim, value_dim, rank, ld;
  float tau, eps;
  __host__ __device__ uint32_t q_cols() const { return heads * dim; }
  __host__ __device__ uint32_t v_cols() const { return heads * value_dim; }
  __host__ __device__ uint32_t cols() const { return 2 * q_cols() + 2 * v_cols() + rank; }
  __host__ __device__ size_t state_floats() const { return (size_t)heads * dim * value_dim; }
};
template <typename T>
struct GlaWeights {
  const T *decay;           // [heads * dim][rank]
  const float *bias, *norm;  // [heads * dim], [value_dim]
};
// Token by token: the sequences of the batch that have at most `most_rows` rows.
template <typename T>
int launch_gla_steps(const float *partial, uint32_t splits, size_t split_stride, GlaShape s, GlaWeights<T> w, float *state, StateBatch sb,
                     uint32_t most_rows, T *out, uint32_t ldo, cudaStream_t stream);
// Prompt portions, kGlaChunk rows at a time: within a chunk the scores of all pairs of rows, between chunks the state.
constexpr uint32_t kGlaChunk = 64;
struct GlaChunk {
  uint32_t row, count, pad0, pad1;  // batch rows [row, row + count) of one sequence
};
struct GlaPortion {
  uint32_t seq, chunk, chunks, pad;  // its chunks follow one another in the list
};
struct GlaPortions {
  const GlaChunk *chunks;
  const GlaPortion *portions;
  uint32_t num_chunks, num_portions;
};
bool gla_chunks_supported(GlaShape s);
// Bytes of scratch that a batch needs (chunk operands, then the heads' outputs in f32).
size_t gla_scratch_bytes(GlaShape s, uint32_t chunks, uint32_t rows);
int launch_gla_chunks(const float *partial, uint32_t splits, size_t split_stride, GlaShape s, GlaWeights<bf16> w, float *state, StateBatch sb,
                      GlaPortions p, void *scratch, bf16 *out, uint32_t ldo, cudaStream_t stream);
int gla_poll_error(uint32_t *code);

// ---- latent attention ---------------------------------------------------------------------
//
// The cache of one layer holds, per token, the normalised latent (kv_rank values) followed by the rotated key
// part that all heads share (rot_dim values): [block][slot][row_stride], row_stride an odd multiple of 8.
struct LatentShape {
  uint32_t heads, dim, rot_dim, value_dim, kv_rank, window, rope_dims, block_size, row_stride;
  float scale, eps;
  bool gated = true;  // the output has a gate per value
  uint32_t ld = 0;    // row stride of the joint projection (0: its columns)
  __host__ __device__ uint32_t q_dim() const { return dim + rot_dim; }
  // Columns of the joint projection: queries, latent + shared key part, output gate.
  __host__ __device__ uint32_t q_cols() const { return heads * (dim + rot_dim); }
  __host__ __device__ uint32_t kv_cols() const { return kv_rank + rot_dim; }
  __host__ __device__ uint32_t out_cols() const { return heads * value_dim; }
  __host__ __device__ uint32_t cols() const { return q_cols() + kv_cols() + (gated ? out_cols() : 0); }
  __host__ __device__ uint32_t row_ld() const { return ld ? ld : cols(); }
  // First position that a query at `pos` sees.
  __host__ __device__ uint32_t first_key(uint32_t pos) const { return KeyRange{window, 0}.first(pos); }
};
// Folds the joint projection's partial sums: queries (rotated) to q [rows][heads][dim + rot_dim], the normalised
// latent and the rotated shared key part to the cache row of the token.
template <typename T>
int launch_latent_prepare(const float *partial, uint32_t splits, size_t split_stride, const float *norm_w, const float *rope_cos,
                          const float *rope_sin, const uint32_t *positions, const uint32_t *slot_block, const uint32_t *slot_slot,
                          T *q, T *cache, LatentShape ls, uint32_t rows, cudaStream_t stream);
// Any shape, any mix of rows: one CTA per (row, head). The query is taken into the latent space (w_uk), the
// weighted latent back out of it (w_uv), and the result is gated: out[r * ldo + h * value_dim + v].
template <typename T>
int launch_latent_attention_generic(const T *q, const T *cache, const T *w_uk, const T *w_uv, const float *gate_partial,
                                    uint32_t splits, size_t split_stride, LatentShape ls, AttnBatch batch, T *out, uint32_t ldo,
                                    cudaStream_t stream);

// Tuned path for rows that decode, one at a time or a few together (bf16; dim, kv_rank and rot_dim multiples of 16):
// `row_list` names the batch rows, and item i of the buffers below belongs to row_list[i].
bool latent_decode_supported(LatentShape ls);
constexpr uint32_t kLatentMaxSplits = 16;
// Pieces the window is cut into so that the batch fills the machine.
uint32_t latent_decode_splits(LatentShape ls, uint32_t rows, uint32_t max_position);
size_t latent_decode_scratch_floats(LatentShape ls, uint32_t rows, uint32_t splits);
// Queries (from launch_latent_prepare) into the latent space: qa [rows][heads][kv_rank + rot_dim].
int launch_latent_absorb(const bf16 *q, const bf16 *w_uk, const uint32_t *row_list, uint32_t rows, bf16 *qa, LatentShape ls,
                         cudaStream_t stream);
// Attention over the cached latents (the rows of this step included), values and gate. `scratch` holds
// latent_decode_scratch_floats floats; first_row as in StateBatch.
int launch_latent_decode(const bf16 *qa, const bf16 *cache, const bf16 *w_uv, const float *gate_partial, uint32_t gate_splits,
                         size_t split_stride, const uint32_t *row_list, const uint32_t *first_row, uint32_t rows, AttnBatch batch,
                         uint32_t splits, float *scratch, LatentShape ls, bf16 *out, uint32_t ldo, cudaStream_t stream);
int latent_poll_error(uint32_t *code);

// Tuned path for prompt portions (bf16; dim, rot_dim and value_dim multiples of 16): keys and values are expanded once
// per token. A portion's rows in the expanded buffers cover its own tokens and those before it that a window reaches.
struct LatentPortion {
  uint32_t seq, row, position, count;  // sequence; first expanded row, the position it stands for, number of rows
};
struct LatentTile {
  uint32_t row_start, num_rows, position;  // batch rows of one sequence, position of the first
  int32_t row_of_zero;                     // expanded row that position 0 of the sequence would have
};
constexpr uint32_t kLatentTileRows = 128;
bool latent_prefill_supported(LatentShape ls);
// Cached latents [rows][kv_rank] and rotated parts [rows][rot_dim] of the portions.
int launch_latent_gather(const bf16 *cache, const uint32_t *tables_flat, const uint32_t *table_offsets, const LatentPortion *portions,
                         uint32_t num_portions, uint32_t longest, bf16 *latents, bf16 *rotated, LatentShape ls, cudaStream_t stream);
// `expanded`: [rows][heads * dim | heads * value_dim], the latents times W_uk and W_uv. The buffers hold
// `rows_capacity` rows of finite values.
int launch_latent_prefill(const bf16 *q, const bf16 *expanded, const bf16 *rotated, uint32_t rows_capacity, const float *gate_partial,
                          uint32_t splits, size_t split_stride, const LatentTile *tiles, uint32_t num_tiles, LatentShape ls, bf16 *out,
                          uint32_t ldo, cudaStream_t stream);
int latent_prefill_poll_error(uint32_t *code);

// ---- mixture of experts ------------------------------------------------------------------------
//
// Every row goes through `top` of the experts, chosen by the largest sigmoid of the router's logits; the score multiplies
// the expert's input. A shared expert (shared_ffn = 0: none) takes every row as it is. An expert is W_down (silu(W_gate x) *
// (W_up x)). Rows are copied into the order of their experts, and the two products run over tiles of rows of one expert.
// Expert weights are stacked: up [experts][2 * ffn][hidden] with gate row f at 2f and up row f at 2f + 1, down
// [experts][hidden][ffn]; the shared expert's the same with one expert.
// Variants: softmax of the logits for the sigmoid; a correction per output of the router that takes part in the choice only;
// `identity` further outputs of the router whose experts return their input (they take no part in the products); scores that
// multiply the experts' outputs (where they are summed: SublayerOutput::weight); other gated activations. groups: the outputs form
// that many groups of neighbours, and only those of the `keep` groups with the largest scores in them can be chosen (scores are not
// negative). renorm: the chosen scores are divided by their sum (+ 1e-20). Experts without a gate (GatedAct::plain) have `up`
// [experts][ffn][hidden].
struct MoeShape {
  uint32_t hidden, experts, top, ffn, shared_ffn;
  uint32_t identity = 0;
  bool softmax = false, weigh_output = false;
  GatedAct act{}, shared_act{};
  uint32_t groups = 0, keep = 0;
  bool renorm = false;
  uint32_t logits_ld = 0;  // row stride of the router's partial sums (0: its outputs)
  __host__ __device__ uint32_t outputs() const { return experts + identity; }
  __host__ __device__ uint32_t row_ld() const { return logits_ld ? logits_ld : outputs(); }
  __host__ __device__ uint32_t up_cols() const { return act.plain() ? ffn : 2 * ffn; }
  __host__ __device__ uint32_t shared_up_cols() const { return shared_act.plain() ? shared_ffn : 2 * shared_ffn; }
};
struct MoeTile {
  uint32_t expert, row, count;  // sorted rows [row, row + count) go through `expert`; count 0: nothing to do
};
struct MoePlan {
  uint32_t tile_rows;             // rows per tile
  uint32_t tiles;                 // entries of the tile list
  uint32_t up_splits, down_splits;  // k splits of the two products
  bool tensor_core;
};
MoePlan moe_plan(bool is_bf16, MoeShape s, uint32_t rows);
constexpr uint32_t kMoeMaxExperts = 1024;
// Device buffers of a step of up to the largest batch.
template <typename T>
struct MoeBuffers {
  uint32_t *chosen = nullptr;  // [rows][top]
  float *score = nullptr;      // [rows][top] (batches of few rows: only with weigh_output)
  uint32_t *histogram = nullptr;  // [moe_histogram_words]
  uint32_t *place = nullptr;   // [rows][top]: sorted row of each choice, kNoPlace for an identity expert
  float *row_score = nullptr;  // [rows * top] by sorted row
  MoeTile *tiles = nullptr;    // [plan.tiles]
  T *x = nullptr;              // [rows * top][hidden] sorted rows
  T *act = nullptr;            // [rows * top][ffn], then [rows][shared_ffn]
  float *up = nullptr;         // k-split products of `up`, moe_up_floats
  float *down = nullptr;       // [splits][rows * top][hidden]
};
size_t moe_histogram_words(MoeShape s, uint32_t rows);
size_t moe_up_floats(bool is_bf16, MoeShape s, uint32_t rows);
// Experts and scores of every row from the router's partial sums [splits][rows][outputs], and the sorted order. correction:
// [outputs], may be null.
template <typename T>
int launch_moe_route(const float *logits, uint32_t splits, size_t split_stride, const float *correction, const T *x, MoeShape s, MoePlan plan,
                     MoeBuffers<T> b, uint32_t rows, cudaStream_t stream);
// Both products: `down` of the sorted rows into b.down, of the shared expert into shared_out [down_splits][rows][hidden].
template <typename T>
int launch_moe_experts(const T *x, const T *w_up, const T *w_down, const T *shared_up, const T *shared_down, MoeShape s, MoePlan plan,
                       MoeBuffers<T> b, float *shared_out, uint32_t rows, cudaStream_t stream);
// One product of the grouped kind on tcgen05: rows of `x` by tile through rows [expert * n, (expert + 1) * n) of `w`, and rows of
// `shared_x` through `shared_w` (shared_n = 0: none). swiglu: activations to act / shared_act (row stride n / 2, shared_n / 2; n, shared_n
// for experts without a gate), the products multiplied by row_score (null = 1); else f32 to out / shared_out, [splits][rows][n].
struct MoeProduct {
  const bf16 *x, *w, *shared_x, *shared_w;
  uint32_t n, k, shared_n, shared_k;
  uint32_t sorted_rows, rows, experts;
  const MoeTile *tiles;
  const float *row_score;
  bf16 *act, *shared_act;
  float *out, *shared_out;
  GatedAct f{}, shared_f{};
};
bool moe_tc_supported(MoeShape s);
int launch_moe_product_tc(const MoeProduct &p, bool swiglu, uint32_t splits, MoePlan plan, cudaStream_t stream);
int moe_poll_error(uint32_t *code);

// ---- tensor-parallel hand-over ---------------------------------------------------

constexpr int kMaxTpWorld = 8;
// Largest batch the fused hand-over takes; larger (prefill-sized) batches are bandwidth-bound
// and go through the library all-reduce.
constexpr uint32_t kTpFusedMaxRows = 256;
// Peer-mapped inboxes of every rank of the tensor-parallel group (index = rank; the entry of
// this rank is its own local pointer). An inbox is [parity 2][sender world][slot_floats] units
// of 8 bytes (one f32 of a partial sum and the epoch of the hand-over that wrote it), followed by
// [parity 2][slot_floats] units for the normalised rows of the two-shot variant.
struct TpPeers {
  uint32_t *inbox[kMaxTpWorld];
  int rank, world;
  uint32_t slot_floats;
  uint64_t wait_limit_ns = 2000000000ull;  // how long a poll for a peer's unit may last before it gives up
};
// All-reduce of the partial sums over ranks and split-K slabs + residual add + RMSNorm for
// `rows` batch rows; every rank ends up with the full residual stream in `hidden` and all
// normalised rows in `out`. The epoch of the call is *epoch_base + epoch_add (epoch_base may be null: epoch_add
// alone); epochs cycle through 1 .. 0xFFFFFFFE, one step per call, and consecutive calls alternate in parity.
// With the base in device memory (advanced by launch_tp_state_bump at the end of a step) a step's launches take
// the same arguments every time, so the step can be replayed as a CUDA graph.
// `two_shot`: reduce-scatter to the owner of each row + all-gather of the normalised rows (only
// the owner of a row then holds its current residual); else every rank reduces every row.
template <typename T>
int launch_tp_allreduce_residual_rmsnorm(const TpPeers &peers, const uint32_t *epoch_base, uint32_t epoch_add, const float *partial, uint32_t splits,
                                         size_t split_stride, float *hidden, const float *norm_w, float eps, T *out,
                                         uint32_t rows, uint32_t hidden_size, bool two_shot, cudaStream_t stream,
                                         uint32_t *ready = nullptr);  // ready: every CTA (one per row) adds 1 when done
// state[0] += epochs (wrapped as described above), state[1] += rows_counted, after the preceding kernel has completed.
int launch_tp_state_bump(uint32_t *state, uint32_t epochs, uint32_t rows_counted, cudaStream_t stream);
int tp_poll_error(uint32_t *code);
// Vocabulary-parallel LM head: `launch_tp_signal` (ranks other than the leader) stores `epoch` into the
// rank's flag in the leader's memory once the preceding kernel of the stream has completed;
// `launch_tp_wait_flags` (leader) holds the stream until the flags of ranks 1 .. world-1 carry `epoch`
// (bounded: after `limit_ns` the hand-over error word gets bit 1 and the stream goes on).
int launch_tp_signal(uint32_t *flag, uint32_t epoch, cudaStream_t stream);
int launch_tp_wait_flags(const uint32_t *flags, uint32_t epoch, int world, uint64_t limit_ns, cudaStream_t stream);
// Launches a kernel whose only thread waits on a barrier that nothing arrives at, with the given
// limit: the bounded wait must give up (timed_out = 1) and the kernel must end normally.
int selftest_bounded_wait(uint64_t limit_us, uint32_t *timed_out, uint32_t *waited_us);
// The same for the peer polls of the tensor-parallel hand-over: one thread polls inbox units that
// nobody writes (both unit formats); each poll must give up after the limit, the device error word
// must be set (and is cleared again), and the kernel must end normally.
int selftest_peer_wait(uint64_t limit_us, uint32_t *timed_out, uint32_t *waited_us);

// ---- GEMM ----------------------------------------------------------------------

// partial[s][r][n] = sum over the k-range of split s of x[r][k] * w[n][k]
// (tensor.rs:114-128 without the bias). x: [rows][k] (row stride ldx),
// w: [n][k] row-major (row stride ldw).
struct GemmPlan {
  uint32_t splits;
  bool tensor_core;     // tcgen05 path (bf16 only)
  bool cluster_reduce;  // the k splits of a tile form a cluster and reduce in shared memory
  uint32_t out_slabs;   // slabs the consumer has to sum: 1 with cluster_reduce, else `splits`
  uint32_t ldc;         // row stride of the output when it is a column block of a wider matrix (0 = n)
};
GemmPlan gemm_plan(bool is_bf16, uint32_t rows, uint32_t n, uint32_t k, uint32_t ldx, uint32_t ldw);
template <typename T>
int launch_gemm(const T *x, uint32_t ldx, const T *w, uint32_t ldw, float *partial, uint32_t rows,
                uint32_t n, uint32_t k, GemmPlan plan, cudaStream_t stream, ReadyWait ready = {});  // `ready`: honoured by the tensor-core path only (GemmPlan::tensor_core)
size_t gemm_partial_floats(bool is_bf16, uint32_t max_rows, uint32_t n, uint32_t k);
// Number of CTAs split-K aims for on small batches (default 296, two per SM).
void gemm_set_target_ctas(uint32_t ctas);
// Ring layout of the decode-batch GEMM: 5 = deep weight ring + short activation ring, 4 = equal rings.
void gemm_set_small_stages(int stages);

// SIMT GEMM: exact k-ascending accumulation per output, no FMA for f32.
template <typename T>
int launch_gemm_simt(const T *x, uint32_t ldx, const T *w, uint32_t ldw, float *out, uint32_t rows,
                     uint32_t n, uint32_t k, cudaStream_t stream);
// tcgen05 / TMEM / TMA GEMM (bf16).
enum GemmEpilogue : uint32_t { kGemmPartials = 0, kGemmSwiglu = 1, kGemmGelu = 2, kGemmStore = 3, kGemmRelu2 = 4, kGemmGeglu = 5 };
bool gemm_tc_supported(uint32_t rows, uint32_t n, uint32_t k, uint32_t ldx, uint32_t ldw,
                       const void *x, const void *w);
int launch_gemm_tc(const bf16 *x, uint32_t ldx, const bf16 *w, uint32_t ldw, float *partial,
                   uint32_t rows, uint32_t n, uint32_t k, uint32_t splits, cudaStream_t stream,
                   bf16 *act = nullptr, bool cluster_reduce = false, uint32_t ldc = 0,
                   ReadyWait ready = {}, GemmEpilogue epi = kGemmPartials, const float *bias = nullptr);
// The same projection with its result stored as bf16 activations, act[r * ld_act + n] = f(x.w_n + bias[n]), f = GELU (tanh
// form), the square of relu or the identity; bias may be null. kGemmGeglu: rows 2f and 2f + 1 of w are gate and up of the same f, and
// act[r * ld_act + f] = GELU(gate) * up. One k split only.
int launch_gemm_act(const bf16 *x, uint32_t ldx, const bf16 *w, uint32_t ldw, bf16 *act, uint32_t ld_act, uint32_t rows, uint32_t n,
                    uint32_t k, GemmEpilogue epi, cudaStream_t stream, const float *bias = nullptr);
// Gate/up projection with SwiGLU in the epilogue: `w_interleaved` is [2 * ffn][k] with gate row f
// at 2f and up row f at 2f + 1; writes act[r][f] = silu(x.gate_f) * (x.up_f) and no partials.
// One k split only (gemm_plan(...).splits == 1 and .tensor_core).
int launch_gemm_swiglu(const bf16 *x, uint32_t ldx, const bf16 *w_interleaved, uint32_t ldw, bf16 *act, uint32_t rows,
                       uint32_t ffn, uint32_t k, cudaStream_t stream, ReadyWait ready = {});
// Device error word set by kernels whose bounded waits ran out (0 = none).
int gemm_tc_poll_error(uint32_t *code);

}  // namespace orion
