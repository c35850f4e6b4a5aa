// Model (weights in the tiled layouts) and session (KV cache, activations, CUDA graph of a step).
#pragma once
#include <map>
#include <set>
#include <string>
#include <vector>

#include "attention.cuh"
#include "common.cuh"
#include "gemv.cuh"

namespace lmb {

enum MapKind { MAP_PLAIN = 0, MAP_QKV = 1, MAP_O = 2, MAP_GATEUP = 3, MAP_DOWN = 4, MAP_STACK = 5 };
constexpr int kMaxSrc = 6;             // logical tensors one internal matrix can hold

// How one internal (tiled) matrix maps onto up to kMaxSrc logical [out,in] tensors of the
// reference (src/NN.jl:330-341, 238-244) -- including the head split f = h + H*d that the
// reference's column-major reshape implies (src/NN.jl:347-354), the GQA mapping q = kv + KV*g
// (src/NN.jl:305-317), the RoPE pairing (d, d + D/2) (src/NN.jl:274-276) and the tensor-parallel
// shard of this rank.
struct WMap {
  int kind = MAP_PLAIN;
  int rows = 0, K = 0;       // internal valid extent
  int RB = 0, KC = 0;        // padded extent in 16-row blocks / 32-k chunks
  int H = 0, KV = 0, D = 0, G = 0, Hl = 0, KVl = 0, kv_off = 0;
  int inter_l = 0, inter_off = 0;
  int src_rows[kMaxSrc] = {0, 0, 0, 0, 0, 0};
  int src_cols[kMaxSrc] = {0, 0, 0, 0, 0, 0};
  // MAP_STACK: tensor s occupies rows row_off[s] .. + src_rows[s] and columns col_off[s] .. + src_cols[s], the rest is zero
  int n_src = 0;
  int row_off[kMaxSrc] = {0, 0, 0, 0, 0, 0};
  int col_off[kMaxSrc] = {0, 0, 0, 0, 0, 0};
  // rows of heads pair_head[s] wide whose first pair_dims[s] features rotate in half-split pairs (i, i + dims / 2): internal rows 2i and
  // 2i + 1 hold pair i.  Applied to queries and keys alike it changes no product, and a pair always sits in neighbouring rows.
  int pair_head[kMaxSrc] = {0, 0, 0, 0, 0, 0};
  int pair_dims[kMaxSrc] = {0, 0, 0, 0, 0, 0};
};

struct LayerWeights {
  void* wqkv = nullptr;
  void* wo = nullptr;
  void* wgu = nullptr;
  void* wdown = nullptr;
  float* attn_norm = nullptr;
  float* ffn_norm = nullptr;
  // Whisper decoder layers only
  void* wq_cross = nullptr;      // encoder_attn.q_proj
  void* wo_cross = nullptr;      // encoder_attn.out_proj
  float* attn_norm_b = nullptr;  // LayerNorm biases
  float* ffn_norm_b = nullptr;
  float* cross_norm = nullptr;
  float* cross_norm_b = nullptr;
  float* b_qkv = nullptr;        // biases in internal row order (k rows zero)
  float* b_o = nullptr;
  float* b_q_cross = nullptr;
  float* b_o_cross = nullptr;
  float* b_fc1 = nullptr;
  float* b_fc2 = nullptr;
  // Whisper, fused step: what folding a LayerNorm into the Linear that follows it needs (InvScale): W g and W b + bias
  // per internal row of q/k/v, of the cross-attention q projection and of fc1
  float *wg_qkv = nullptr, *bf_qkv = nullptr, *wg_qc = nullptr, *bf_qc = nullptr, *wg_fc1 = nullptr, *bf_fc1 = nullptr;
};

// One layer of a decoder whose layers are described one by one (LMB200_ARCH_LAYERED, csrc/layered.cu): its sizes and
// constants, and how its tensors are stacked into the matrices the step multiplies with.
struct LayerSpec {
  lmb200_layer_config c{};
  std::vector<double> decay;
  // input projections, all reading the same vector: latent attention [dq | dkv | g | up], retention [q | k | v | g | up], attention
  // [q | k | v], channel delta [q | k | v | b | a1 | g1], lightning [q | k | v | g].
  // Every part starts on a multiple of 32 rows.  The first n_store rows are mixer inputs, the rest the feed-forward's.
  WMap m_in;
  int row0[kMaxSrc] = {0, 0, 0, 0, 0, 0};
  int n_store = 0;
  WMap m_uq, m_ukv;          // latent attention: queries from their latent; [uk | uv], per-head keys and values from the latent
  WMap m_out;                // [o | down] side by side: mixer output columns from 0, feed-forward columns from cat0
  int cat0 = 0;
  // LMB200_BLOCK_POSTNORM: feed-forward, token input
  WMap m_gu, m_down, m_sg, m_sp;
  WMap m_lr;                 // channel delta: [a2 over the a1 columns; g2 over the g1 columns]
  int lr_g1 = 0;             // column of g1's output in m_lr's input
  int k_ld = 0, v_ld = 0;    // attention: cached key and value rows (widths rounded up to 8, the gap zero)
  int lat_rot = 0, lat_ld = 0;   // latent cache row: latent from 0, rotated key part from lat_rot, lat_ld elements in all
};
struct LayeredWeights {
  void *w_in = nullptr, *w_out = nullptr, *w_uq = nullptr, *w_ukv = nullptr;
  void *w_ukt = nullptr, *w_uv = nullptr;     // row-major [heads, kv_rank, dim] and [heads * vdim, kv_rank] (absorbed attention)
  float *norm = nullptr, *q_norm = nullptr, *kv_norm = nullptr;
  void *w_gu = nullptr, *w_down = nullptr, *w_sg = nullptr, *w_sp = nullptr, *w_lr = nullptr;
  float *norm2 = nullptr, *side_norm = nullptr, *mix_norm = nullptr;
  float *conv = nullptr;                      // channel delta: [taps][channels of q | k | v], tap 0 meets the current token
  float *a_log = nullptr, *dt_bias = nullptr;
  float *inv_freq = nullptr;                  // [rot_dims / 2]
  int rot_id = -1;                            // layers with the same frequencies share an angle table (Model::rot_freqs)
  float *decay = nullptr;                     // retention: [heads][kDecayPow]: decay^0 .. decay^(kDecayPow - 1)
};
constexpr int kDecayPow = 136;

struct Model {
  bool tp_solo = false;        // profiling aid: shard of one rank, no all-reduce
  uint32_t magic = 0x4D4F444C;
  Ctx* ctx = nullptr;
  lmb200_model_config cfg{};
  int esz = 4;
  int Hl = 0, KVl = 0, G = 0, D = 0, kv_off = 0, inter_l = 0, inter_off = 0;
  WMap m_qkv, m_o, m_gu, m_down, m_head;
  WMap m_qc;                    // Whisper: cross-attention q projection (q rows only)
  float* final_norm_b = nullptr;
  float* pos_emb = nullptr;     // Whisper: [max_positions, hidden] float32
  void* embed_tiled = nullptr;  // Whisper: the embedding table in GEMV layout (tied head)
  float *wg_head = nullptr, *bf_head = nullptr;   // Whisper, fused step: the final LayerNorm folded into the head
  bool fold_valid = false;      // the folded vectors match the weights (set_weight / init_random clear it)
  std::vector<LayerWeights> layers;
  void* embed = nullptr;        // [vocab, hidden] row-major, model dtype
  float* final_norm = nullptr;
  void* lm_head = nullptr;
  float* inv_freq = nullptr;    // [D/2]
  int64_t weight_bytes = 0;
  // LMB200_ARCH_LAYERED
  std::vector<LayerSpec> specs;
  std::vector<LayeredWeights> lw;
  float softcap = 0.f, embed_scale = 1.f;
  int block = 0, side_dim = 0;
  bool tied_head = false;
  void* side_embed = nullptr;   // [vocab, n_layers * side_dim], model dtype
  std::vector<std::vector<float>> rot_freqs;   // the distinct frequency lists of the layers
  std::set<std::string> weights_set;   // registry names given through lmb200_model_set_weight
  bool all_weights_set = false;        // lmb200_model_init_random filled everything
};

struct Session {
  uint32_t magic = 0x53455353;
  Model* m = nullptr;
  int B = 0, max_ctx = 0, cap = 0;
  int host_pos = 0;               // the furthest position of any sequence (bounds checks)
  std::vector<int> host_pos_v;    // the host's copy of the per-sequence positions
  bool ragged = false;            // the positions differ: kernels take the per-sequence RoPE path
  bool in_ragged_prefill = false; // steps of lmb200_prefill_ragged: the host positions are set at its end
  int* limit = nullptr;           // device [B]: a sequence at its limit does not advance
  float* ragged_logits = nullptr; // [B][logits_pitch]: each sequence's logits at its own last prompt position
  // cache: [L][B][KVl][cap/16][32*D]
  void* kv = nullptr;
  int64_t kv_head_stride = 0, kv_batch_stride = 0, kv_layer_stride = 0;
  // activations
  float* x = nullptr;
  float* delta = nullptr;
  float* logits = nullptr;
  void* xn = nullptr;
  void* qbuf = nullptr;
  void* attn_out = nullptr;
  void* act = nullptr;
  int Bp = 0;                   // batch padding of the tiled activation buffers (8, 16 or 32)
  int q_pitch = 0, logits_pitch = 0;
  int* tokens = nullptr;
  int* pos = nullptr;           // device [B]: one position per sequence
  int* step_ctr = nullptr;
  int* stop = nullptr;          // [0] end-of-text id or -1, [1] sequences that produced it, [2 + b] sequence b did
  int* tok_hist = nullptr;      // [cap][B]
  int* prompt = nullptr;        // staging for prefill
  int64_t prompt_cap = 0;
  // scratch
  float* gemv_partials = nullptr;
  unsigned* gemv_counters = nullptr;
  float* part_o = nullptr;
  float* part_ml = nullptr;
  unsigned* attn_counters = nullptr;   // [B*KVl], zero between launches
  float* sum_slots = nullptr;          // fused Whisper step: per-CTA sums of x beside ssq (LayerNorm's mean)
  void* prefill_buf = nullptr;         // scratch of the GEMM prompt phase, kept between prompts
  int64_t prefill_bytes = 0;
  int keys_per_cta = 0, nsplit = 0;
  GemvPlan p_qkv, p_o, p_gu, p_down, p_head, p_qc;
  // Whisper: cross-attention cache [L][B][H][cross_cap/16][32*D] and its split plan
  void* cross_kv = nullptr;
  int cross_cap = 0;
  int64_t cross_head_stride = 0, cross_batch_stride = 0, cross_layer_stride = 0;
  int cross_keys_per_cta = 0, cross_nsplit = 0;
  // fused step (bf16 Llama): the row-parallel projections do the all-reduce, the residual add and the
  // RMSNorm preparation in their epilogue, the other projections apply the norm's scale in theirs
  bool fused = false;
  float* xT = nullptr;          // residual stream [hidden][Bp] float32 (batch fastest)
  float* ssq = nullptr;         // [256][32] per-CTA sums of squares of the residual rows
  int embed_rows_per_cta = 32;
  float* capture = nullptr;     // [L][B][hidden] when enabled
  bool capture_on = false;
  // Tensor parallelism, fused step: every rank multiplies only its slice of the (replicated) head's rows and the ranks
  // exchange their (best logit, token id) pairs; the full logits are computed only when a caller asks for them
  bool head_sliced = false;
  int head_rg0 = 0, head_rows = 0;      // this rank's first 128-row group and its valid rows
  GemvPlan p_head_slice;
  float* logits_slice = nullptr;        // [B][head_pitch] float32
  int head_pitch = 0;
  cudaGraphExec_t graph_full = nullptr;   // head and logits
  cudaGraphExec_t graph_body = nullptr;   // no head
  cudaGraphExec_t graph_tok = nullptr;    // sliced head, tokens only (head_sliced)
  cudaStream_t graph_stream = nullptr;
  int graph_nodes_full = 0, graph_nodes_body = 0, graph_nodes_tok = 0;
  // LMB200_ARCH_LAYERED (csrc/layered.cu): per layer a latent cache [B][cap][lat_ld], a recurrent state
  // [B][heads][dim][round_up(vdim, 4)] float32, or NULL (a layer that reads another layer's latent cache)
  // attention: keys [B][kv_heads][cap][k_ld] and values [B][kv_heads][cap][v_ld]; channel delta also the last raw inputs of its
  // convolutions, position p in slot p % taps of [B][taps][channels] float32
  std::vector<void*> latent, keys, values;
  std::vector<float*> state, conv;
  struct LayeredScratch* lay = nullptr;
  // a batch above 32: this session owns nothing on the device, it is a row of sub-sessions of at most 32 sequences
  std::vector<uint64_t> parts;
};

// the entry points of a session of more than 32 sequences (csrc/wide.cu): each runs the sub-sessions in turn
int32_t wide_create(Model* M, int batch, int max_ctx, lmb200_session* out);
int32_t wide_destroy(Session* S);
int32_t wide_reset(Session* S);
int32_t wide_position(Session* S, int32_t* pos);
int32_t wide_set_position(Session* S, int32_t pos);
int32_t wide_set_positions(Session* S, const int32_t* pos);
int32_t wide_positions(Session* S, int32_t* pos_out);
int32_t wide_fill_kv_random(Session* S, int32_t n_pos, uint64_t seed);
int32_t wide_set_capture(Session* S, int32_t enable);
int32_t wide_read_layer_output(Session* S, int32_t layer, float* host);
int32_t wide_prefill(Session* S, const int32_t* tokens, int32_t n, float* logits_out);
int32_t wide_prefill_ragged(Session* S, const int32_t* tokens, const int32_t* lengths, int32_t n_max, float* logits_out);
int32_t wide_extend(Session* S, const int32_t* tokens, const int32_t* lengths, int32_t n_want, const int32_t* want, float* logits_out);
int32_t wide_decode_step(Session* S, const int32_t* tokens_in, int32_t* next_tokens_out, float* logits_out);
int32_t wide_decode_n(Session* S, const int32_t* first_tokens, int32_t n_steps, int32_t* tokens_out);
int32_t wide_decode_until(Session* S, const int32_t* first_tokens, int32_t max_steps, int32_t eot_token, int32_t* tokens_out,
                          int32_t* steps_done);
int32_t wide_step_bytes(Session* S, int32_t T, int64_t* bytes);

int32_t step_kernels_configure();

// decoders described layer by layer (csrc/layered.cu): what the model and session entry points hand over to
void layered_free_model(Model* M);
int32_t layered_init_random(Model* M, uint64_t seed, float sigma);
int32_t layered_set_weight(Model* M, const char* name, const float* host, int32_t rank, const int64_t* dims, int32_t layout);
std::vector<std::string> layered_weight_names(const Model* M);
int32_t layered_session_create(Model* M, int batch, int max_ctx, lmb200_session* out);
void layered_session_free(Session* S);
// sequences whose position goes back to 0 start from an empty state; a position other than 0 or the present one needs
// `forced` (synthetic contexts) where the model has recurrent layers
int32_t layered_check_positions(const Session* S, const int32_t* pos);
int32_t layered_clear_state(Session* S, const int32_t* new_pos);
int32_t layered_fill_random(Session* S, int32_t n_pos, uint64_t seed);
bool layered_has_state(const Model* M);
int32_t layered_enqueue_step(Session* S, cudaStream_t st, bool with_head);
// the next lengths[b] >= 0 tokens of every sequence (packed), logits of the packed places want[0 .. n_want) (logits_out may be
// NULL).  greedy: want holds every sequence's last place, and the best tokens there become the next step's input
int32_t layered_extend(Session* S, const int32_t* tokens, const int32_t* lengths, int32_t n_want, const int32_t* want, float* logits_out,
                       bool greedy = false);
int64_t layered_step_bytes(const Session* S, int32_t T);
int32_t layered_configure();

// pieces of model.cu and prefill.cu that layered.cu builds on
struct FillSrc {
  uint64_t key[kMaxSrc];
  const float* src[kMaxSrc];     // staged logical tensors (NULL -> generator)
  int colmajor;
  int only_slot;           // -1: all
  float scale;             // sigma / 131072
};
int32_t fill_tiled_dt(Model* M, void* dst, const WMap& m, const FillSrc& f);
// head > 0: every block of `head` rows is stored transposed, [rows / head, cols, head]
int32_t fill_plain_dt(Model* M, int dtype, void* dst, int64_t rows, int64_t cols, uint64_t key, const float* src, int colmajor, float scale,
                      float offset, int head = 0);
int32_t check_weight_shape(const char* name, int32_t rank, const int64_t* dims, int64_t rows, int64_t cols);
int64_t tiled_elems(const WMap& m, int dtype);
void finish_map(WMap& m);
int32_t dmalloc(void** p, int64_t bytes, bool zero, cudaStream_t st);
int32_t push_positions(Session* S);
int32_t embed_prep_launch(Session* S, const float* gain, cudaStream_t st, float scale = 1.0f);
GemvParams gemv_params(Session* S, const void* W, const WMap& m, const GemvPlan& pl, const void* x);
int32_t argmax_launch(Session* S, cudaStream_t st);       // greedy tokens of S->logits into S->tokens
int32_t advance_launch(Session* S, cudaStream_t st);      // end of a step on one GPU
int32_t run_step(Session* S, bool with_head, bool want_logits = true);

// Destination of a run of output rows of a GEMM over many tokens: element (token t, row row0 + r), r < rows, goes to
// dst[t * pitch + r] after the activation.
enum RowSegKind {
  SEG_F32 = 0,        // float32
  SEG_ACT = 1,        // model dtype
  SEG_RELU2 = 2,      // relu(v)^2, model dtype
  SEG_SILU = 3,       // silu(v), model dtype
  SEG_SOFTCAP = 4,    // softcap * tanh(v / softcap), float32 (softcap 0: v)
  SEG_ROT = 5,        // bf16: neighbouring rows (2i, 2i + 1) of every head are rotated by angle i of the token's table row
  SEG_SIGMOID = 6,    // sigmoid(v), model dtype
  SEG_DECAY = 7,      // -exp(rate[r / head]) softplus(v + bias[r]), float32
  SEG_GELU_TOKEN = 8  // gelu(v) * table[tokens[t] * table_pitch + r], model dtype
};
struct RowSeg {
  int row0 = 0, rows = 0, kind = SEG_F32, pitch = 0;
  void* dst = nullptr;
  // SEG_ROT: heads of rot_head rows, features rot_off .. rot_off + rot_dims - 1 rotate (all even); rot[token * rot_dims / 2 + i] = (cos, sin)
  const float2* rot = nullptr;
  int rot_head = 0, rot_off = 0, rot_dims = 0;
  const float *rate = nullptr, *bias = nullptr;        // SEG_DECAY
  int head = 1;
  const void* table = nullptr;                         // SEG_GELU_TOKEN: model dtype, table_rows tokens
  const int* tokens = nullptr;
  int table_pitch = 0, table_rows = 0;
};
constexpr int kMaxSegs = 6;
struct RowSegs {
  RowSeg s[kMaxSegs];
  int n = 0;
  float softcap = 0.f;
  void add(int row0, int rows, int kind, void* dst, int pitch) { s[n].row0 = row0; s[n].rows = rows; s[n].kind = kind; s[n].dst = dst; s[n].pitch = pitch; ++n; }
};
// rows of W (bf16 weight layout) times X [T, ldx] row-major bf16 (columns past K are not read), each row to its segment
int32_t gemm_segments_bf16(Ctx* ctx, const void* W, const void* X, int ldx, int T, int rows, int K, const RowSegs& segs, cudaStream_t st);
// act[t * ld_act + i] = silu(gate_i) up_i over MAP_GATEUP rows (bf16), i < n_act
int32_t gemm_silu_gate_bf16(Ctx* ctx, const void* W, const void* X, int ldx, int T, int rows, int K, void* act, int ld_act, int n_act, cudaStream_t st);
// prompt phase as GEMMs + flash attention (csrc/prefill.cu)
int32_t prefill_configure();
bool prefill_gemm_ok(const Session* S, int n);
// lens_dev: NULL (every sequence has n tokens) or device [B] prompt lengths <= n (the last-position rows are taken per sequence)
int32_t prefill_gemm(Session* S, const int* tokens_dev, int n, const int* lens_dev, cudaStream_t st);
int32_t prefill_linear(Ctx* ctx, const void* W, const float* x_dev, int T, int rows, int K, float* out_dev, cudaStream_t st);
Model* model_from(lmb200_model h);
Session* session_from(lmb200_session h);

}  // namespace lmb
