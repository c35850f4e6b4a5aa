// Decoders described layer by layer (LMB200_ARCH_LAYERED): the layers' specifications, their weights, the per-layer caches and
// states of a session, and the two ways a step runs.
//   fused step   bf16 decoding, one token per sequence, captured in a CUDA graph: GEMVs whose epilogues carry the norm's scale,
//                the feed-forward's activation, the residual sum and the next norm's preparation.  A layer's projections are
//                one matrix, and so are the two output projections of a parallel block: retention takes three launches, latent
//                attention seven.  Where the sublayers are normed on their output (LMB200_BLOCK_POSTNORM) the output projections
//                apply that norm themselves (EPI_POST_NORM): mixer 3 launches (channel delta 4), feed-forward 2, token input 2.
//   rows step    any number of tokens of any sequences, packed: prompts, portions of prompts, mixed calls; and every
//                float32 step.
#include <math.h>
#include <stdio.h>
#include <string.h>

#include <algorithm>

#include "activations.cuh"
#include "delta.cuh"
#include "latent.cuh"
#include "model.cuh"
#include "pdl.cuh"
#include "retention.cuh"
#include "window_attn.cuh"

namespace lmb {

bool flash_tc_split_supported(int dn, int dr, int dv);
int32_t flash_tc_launch_split(Ctx* ctx, void* out, const void* q, const void* k, const void* kr, const void* v, const FlashSplitView& f, int64_t B,
                              int64_t Sq, int64_t Sk, float scale, cudaStream_t stream);
bool flash_tc_window_supported(int dn, int dv);
int32_t flash_tc_launch_window(Ctx* ctx, void* out, const void* q, const void* k, const void* v, const FlashWindowView& f, int64_t B, int64_t Sq,
                               int64_t Sk, float scale, cudaStream_t stream);

// device buffers of a rows step over up to `cap_T` tokens
struct RowsBuf {
  int64_t cap_T = 0;
  void* base = nullptr;
  int64_t bytes = 0;
  float *x = nullptr, *delta = nullptr, *proj = nullptr;
  void *xn = nullptr, *xq = nullptr, *q = nullptr, *qa = nullptr, *cat = nullptr, *packed = nullptr;
  void *act = nullptr, *side = nullptr, *lr_in = nullptr, *gate = nullptr;      // feed-forward, token input, channel delta's low ranks and gate
  float *beta = nullptr, *log_g = nullptr, *rq = nullptr, *rk = nullptr;        // channel delta
  float* ssq = nullptr;                                                         // lightning: sums of squares per token and head
  float2* angles = nullptr;     // [Model::rot_freqs][cap_T][max_half] (cos, sin) of the tokens' positions
  int max_half = 0;
  std::vector<bool> angles_valid;
  int packed_layer = -1;        // whose latent rows `packed` holds in this step
  int* meta = nullptr;          // tokens | seq | pos | last (sequence whose last token this is, or -1), cap_T each; then start | len | pos0, B each; want
};

struct LayeredScratch {
  // fused step
  float *proj = nullptr, *qf = nullptr;
  void *xq = nullptr, *qa = nullptr;
  std::vector<GemvPlan> p_in, p_out, p_uq;
  int *iota = nullptr, *ones = nullptr;          // [B]
  std::vector<LatentAttnPlan> attn;              // per layer, one token per sequence at the session's capacity
  float* attn_part = nullptr;
  std::vector<WindowPlan> win;                   // the same for attention layers
  unsigned *win_cnt = nullptr, *prompt_cnt = nullptr;
  int64_t prompt_cnt_n = 0;
  std::vector<GemvPlan> p_gu, p_down, p_sg, p_sp, p_lr;
  void *act_ff = nullptr, *act_side = nullptr, *lr_in = nullptr, *qw = nullptr;   // GEMV inputs; prepared queries (CUDA-core attention)
  float *lr = nullptr, *mix_ssq = nullptr, *post_slots = nullptr;                 // post_slots: [3][kPushMaxCtas][32]
  RowsBuf step, prompt;                          // float32 decode step; everything longer
  float* want_logits = nullptr;
  void* want_xn = nullptr;
  int64_t want_cap = 0;
  float* prompt_part = nullptr;                  // partial results of the absorbed attention in a rows step
  int64_t prompt_part_floats = 0;
  void* expanded = nullptr;                      // keys and values multiplied out of the latents (long portions)
  int64_t expanded_bytes = 0;
};

namespace {

constexpr int kChunkMin = 8, kTcMin = 80;   // longest portion from which retention (and the delta rule) runs in chunks of 64, of 128 tokens
constexpr int kDeltaTcMin = 48;         // longest portion from which the delta rule runs on tcgen05
constexpr int kFlashMin = 32;           // shortest portion whose context is expanded to keys and values
constexpr int kBlockTokens = 2048;      // tokens per round of the absorbed attention in a rows step (bounds its scratch)
constexpr uint64_t kIdLayered = 0x200000, kIdLayeredState = 0x300000;
enum LatentSlot { L_DQ = 0, L_DKV = 1, L_G = 2, L_UP = 3 };
enum RetentionSlot { R_Q = 0, R_K = 1, R_V = 2, R_G = 3, R_UP = 4 };
enum DeltaSlot { D_Q = 0, D_K = 1, D_V = 2, D_B = 3, D_A1 = 4, D_G1 = 5 };      // attention: the first three

bool is_latent(const LayerSpec& s) { return s.c.mixer == LMB200_MIXER_LATENT_ATTENTION; }
bool is_attention(const LayerSpec& s) { return s.c.mixer == LMB200_MIXER_ATTENTION; }
bool is_delta(const LayerSpec& s) { return s.c.mixer == LMB200_MIXER_CHANNEL_DELTA; }
bool is_lightning(const LayerSpec& s) { return s.c.mixer == LMB200_MIXER_LIGHTNING; }
bool has_state(const LayerSpec& s) { return !is_latent(s) && !is_attention(s); }
bool post_norm(const Model* M) { return M->block == LMB200_BLOCK_POSTNORM; }
int delta_channels(const LayerSpec& s) { return 2 * s.c.kv_heads * s.c.dim + s.c.heads * s.c.vdim; }
int out_width(const LayerSpec& s) { return s.c.heads * s.c.vdim; }
int q_width(const LayerSpec& s) { return s.c.heads * (s.c.dim + s.c.rot_dim); }
int state_ld(const LayerSpec& s) { return (int)round_up(s.c.vdim, 4); }
int row_ld(int n) { return (int)round_up(n, 8); }
const LayerSpec& cache_spec(const Model* M, int l) { return M->specs[M->specs[l].c.kv_from >= 0 ? M->specs[l].c.kv_from : l]; }
int cache_layer(const Model* M, int l) { return M->specs[l].c.kv_from >= 0 ? M->specs[l].c.kv_from : l; }

int32_t check_layer(const lmb200_layer_config& c, const std::vector<LayerSpec>& before, int i, int block) {
  const bool latent = c.mixer == LMB200_MIXER_LATENT_ATTENTION, attention = c.mixer == LMB200_MIXER_ATTENTION;
  const bool retention = c.mixer == LMB200_MIXER_RETENTION, lightning = c.mixer == LMB200_MIXER_LIGHTNING;
  LMB_REQUIRE(c.mixer >= LMB200_MIXER_LATENT_ATTENTION && c.mixer <= LMB200_MIXER_LIGHTNING, "layer %d: mixer %d", i, c.mixer);
  LMB_REQUIRE((block == LMB200_BLOCK_PARALLEL) == (latent || retention), "layer %d: mixer %d is not built for this arrangement of a layer", i, c.mixer);
  LMB_REQUIRE(c.heads >= 1 && c.dim >= 1 && c.vdim >= 1 && c.ff >= 0, "layer %d: non-positive size", i);
  LMB_REQUIRE(c.ff == 0 || c.ff_kind == (block == LMB200_BLOCK_PARALLEL ? LMB200_FF_RELU2 : LMB200_FF_SILU_GATE), "layer %d: feed-forward of kind %d", i, c.ff_kind);
  LMB_REQUIRE(c.rot_layout == LMB200_ROT_HALF || c.rot_layout == LMB200_ROT_INTERLEAVED, "layer %d: rot_layout %d", i, c.rot_layout);
  LMB_REQUIRE(c.rot_dims >= 0 && c.rot_dims % 2 == 0 && (c.rot_dims == 0 || c.rot_base > 0), "layer %d: rotation of %d features, base %g", i,
              c.rot_dims, c.rot_base);
  if (latent) {
    LMB_REQUIRE(c.q_rank >= 1 && c.kv_rank >= 1 && c.rot_dim >= 0 && c.rot_dims <= c.rot_dim, "layer %d: ranks %d, %d, rotated %d of %d", i,
                c.q_rank, c.kv_rank, c.rot_dims, c.rot_dim);
    LMB_REQUIRE(c.dim <= 1024 && c.kv_rank <= 1024, "layer %d: head width %d, latent width %d (at most 1024)", i, c.dim, c.kv_rank);
    LMB_REQUIRE(c.kv_from < i, "layer %d: kv_from %d is not an earlier layer", i, c.kv_from);
    if (c.kv_from >= 0) {
      const lmb200_layer_config& f = before[c.kv_from].c;
      LMB_REQUIRE(f.mixer == c.mixer && f.kv_from < 0 && f.kv_rank == c.kv_rank && f.rot_dim == c.rot_dim && f.rot_dims == c.rot_dims &&
                      f.rot_base == c.rot_base && f.rot_layout == c.rot_layout,
                  "layer %d: layer %d has no latent cache of its own with the same widths and rotation", i, c.kv_from);
    }
    return LMB200_OK;
  }
  if (attention || c.mixer == LMB200_MIXER_CHANNEL_DELTA)
    LMB_REQUIRE(c.kv_heads >= 0 && (c.kv_heads == 0 || c.heads % c.kv_heads == 0), "layer %d: %d heads over %d key heads", i, c.heads, c.kv_heads);
  if (attention) {
    LMB_REQUIRE(c.rot_dims <= c.dim && c.dim <= 4096 && c.vdim <= 4096, "layer %d: heads of %d x %d, %d features rotated", i, c.dim, c.vdim, c.rot_dims);
    LMB_REQUIRE(c.window >= 0 && c.score_cap >= 0.f && c.scale > 0.f, "layer %d: window %d, score_cap %g, scale %g", i, c.window, c.score_cap, c.scale);
    LMB_REQUIRE(c.rot_factor == 0.0 || (c.rot_factor > 0.0 && c.rot_original > 0.0 && c.rot_fast > 0.0 && c.rot_slow > 0.0 && c.rot_base > 1.0),
                "layer %d: rotation scaled by %g", i, c.rot_factor);
    LMB_REQUIRE(c.kv_from < i, "layer %d: kv_from %d is not an earlier layer", i, c.kv_from);
    if (c.kv_from >= 0) {
      const lmb200_layer_config& f = before[c.kv_from].c;
      LMB_REQUIRE(f.mixer == c.mixer && f.kv_from < 0 && f.kv_heads == (c.kv_heads ? c.kv_heads : c.heads) && f.dim == c.dim && f.vdim == c.vdim,
                  "layer %d: layer %d has no keys and values of its own with the same head count and widths", i, c.kv_from);
    }
    return LMB200_OK;
  }
  if (c.mixer == LMB200_MIXER_CHANNEL_DELTA) {
    LMB_REQUIRE(c.dim <= 256 && c.vdim <= 256, "layer %d: heads of %d x %d (at most 256)", i, c.dim, c.vdim);
    LMB_REQUIRE(c.conv >= 1 && c.conv <= 16 && c.decay_rank >= 1 && c.gate_rank >= 1, "layer %d: %d taps, ranks %d and %d", i, c.conv, c.decay_rank, c.gate_rank);
    return LMB200_OK;
  }
  LMB_REQUIRE(c.decay, "layer %d: no decay", i);
  LMB_REQUIRE(c.rot_dims <= c.dim && c.dim <= 2048 && c.vdim <= 4096, "layer %d: heads of %d x %d, %d features rotated", i, c.dim, c.vdim, c.rot_dims);
  LMB_REQUIRE(!lightning || c.rot_dims == 0, "layer %d: a lightning layer has no rotation", i);
  for (int h = 0; h < c.heads; ++h)
    LMB_REQUIRE(c.decay[h] > 0.0 && c.decay[h] <= 1.0, "layer %d: decay %g of head %d", i, c.decay[h], h);
  return LMB200_OK;
}

// frequencies of the rotated pairs; with rot_factor the slow ones are stretched (YaRN)
std::vector<float> rotation_freqs(const lmb200_layer_config& c) {
  std::vector<float> f(c.rot_dims / 2);
  const double kPi = 3.14159265358979323846, n = c.rot_dims, ln_base = log(c.rot_base);
  auto turns = [&](double t) { return n * log(c.rot_original / (2.0 * kPi * t)) / (2.0 * ln_base); };     // the feature that turns t times
  double lo = 0.0, hi = 0.0;
  if (c.rot_factor > 0.0) {
    lo = std::max(floor(turns(c.rot_fast)), 0.0);
    hi = std::min(ceil(turns(c.rot_slow)), n - 1.0);
  }
  for (int i = 0; i < c.rot_dims / 2; ++i) {
    double x = pow(c.rot_base, -2.0 * i / n);
    if (c.rot_factor > 0.0) {
      const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
      x = x / c.rot_factor * ramp + x * (1.0 - ramp);
    }
    f[i] = (float)x;
  }
  return f;
}
float rotation_scale(const lmb200_layer_config& c) { return c.rot_factor > 0.0 ? (float)(0.1 * log(c.rot_factor) + 1.0) : 1.0f; }

void stack(WMap& m, int slot, int row0, int rows, int col0, int cols) {
  m.row_off[slot] = row0; m.src_rows[slot] = rows; m.col_off[slot] = col0; m.src_cols[slot] = cols;
  if (m.n_src <= slot) m.n_src = slot + 1;
}

void plain_map(WMap& m, int rows, int K) {
  m.kind = MAP_PLAIN; m.rows = rows; m.K = K; m.src_rows[0] = rows; m.src_cols[0] = K;
  finish_map(m);
}

void derive_layer(LayerSpec& s, int width, int block, int side_dim) {
  const lmb200_layer_config& c = s.c;
  s.m_in.kind = s.m_out.kind = s.m_uq.kind = s.m_ukv.kind = s.m_lr.kind = MAP_STACK;
  int at = 0;
  auto part = [&](int slot, int rows) {
    s.row0[slot] = at;
    stack(s.m_in, slot, at, rows, 0, width);
    at += (int)round_up(rows, 32);
  };
  if (is_latent(s)) {
    part(L_DQ, c.q_rank);
    if (c.kv_from < 0) part(L_DKV, c.kv_rank + c.rot_dim);
    part(L_G, c.heads);
    s.n_store = at;
    if (c.ff) part(L_UP, c.ff);
    stack(s.m_uq, 0, 0, q_width(s), 0, c.q_rank);
    s.m_uq.rows = q_width(s); s.m_uq.K = c.q_rank;
    const int uv0 = (int)round_up(c.heads * c.dim, 32);
    stack(s.m_ukv, 0, 0, c.heads * c.dim, 0, c.kv_rank);
    stack(s.m_ukv, 1, uv0, out_width(s), 0, c.kv_rank);
    s.m_ukv.rows = uv0 + out_width(s); s.m_ukv.K = c.kv_rank;
    finish_map(s.m_uq);
    finish_map(s.m_ukv);
    s.lat_rot = (int)round_up(c.kv_rank, 8);
    s.lat_ld = (int)round_up(s.lat_rot + c.rot_dim, 8);
  } else if (is_attention(s)) {
    part(D_Q, c.heads * c.dim);
    if (c.kv_from < 0) {
      part(D_K, c.kv_heads * c.dim);
      part(D_V, c.kv_heads * c.vdim);
    }
    s.n_store = at;
    s.k_ld = row_ld(c.dim);
    s.v_ld = row_ld(c.vdim);
  } else if (is_delta(s)) {
    part(D_Q, c.kv_heads * c.dim);
    part(D_K, c.kv_heads * c.dim);
    part(D_V, out_width(s));
    part(D_B, c.heads);
    s.n_store = at;                             // what follows is the input of the low-rank products
    part(D_A1, c.decay_rank);
    part(D_G1, c.gate_rank);
    s.lr_g1 = (int)round_up(c.decay_rank, 32);
    const int g0 = (int)round_up(c.heads * c.dim, 32);
    stack(s.m_lr, 0, 0, c.heads * c.dim, 0, c.decay_rank);
    stack(s.m_lr, 1, g0, out_width(s), s.lr_g1, c.gate_rank);
    s.m_lr.rows = g0 + out_width(s); s.m_lr.K = s.lr_g1 + c.gate_rank;
    finish_map(s.m_lr);
  } else {
    part(R_Q, c.heads * c.dim);
    part(R_K, c.heads * c.dim);
    if (c.rot_layout == LMB200_ROT_HALF)
      for (int slot : {(int)R_Q, (int)R_K}) { s.m_in.pair_head[slot] = c.dim; s.m_in.pair_dims[slot] = c.rot_dims; }
    part(R_V, out_width(s));
    part(R_G, out_width(s));
    s.n_store = at;
    if (c.ff && block == LMB200_BLOCK_PARALLEL) part(R_UP, c.ff);
  }
  s.m_in.rows = at > 1024 ? (int)round_up(at, 256) : at;        // whole row pairs for the prompt GEMM
  s.m_in.K = width;
  s.cat0 = (int)round_up(out_width(s), 32);
  stack(s.m_out, 0, 0, width, 0, out_width(s));
  s.m_out.rows = width; s.m_out.K = out_width(s);
  if (c.ff && block == LMB200_BLOCK_PARALLEL) {
    stack(s.m_out, 1, 0, width, s.cat0, c.ff);
    s.m_out.K = s.cat0 + c.ff;
  }
  finish_map(s.m_in);
  finish_map(s.m_out);
  if (block == LMB200_BLOCK_PARALLEL) return;
  if (c.ff) {
    WMap& g = s.m_gu;
    g.kind = MAP_GATEUP; g.rows = 16 * (int)ceil_div(c.ff, 8); g.K = width; g.inter_l = c.ff;
    for (int i = 0; i < 2; ++i) { g.src_rows[i] = c.ff; g.src_cols[i] = width; }
    finish_map(g);
    plain_map(s.m_down, width, c.ff);
  }
  if (side_dim) {
    plain_map(s.m_sg, side_dim, width);
    plain_map(s.m_sp, width, side_dim);
  }
}

// where a tensor lives: a slot of a stacked matrix, a float32 vector, the embedding, and / or a row-major copy
struct Target {
  void* tiled = nullptr;
  const WMap* map = nullptr;
  int slot = 0;
  void* plain = nullptr;         // row-major copy in the model dtype (float32 for vectors)
  bool vec = false;
  float offset = 1.f;            // what generated values of a vector lie around
  int head = 0;                  // the copy holds heads of this many rows transposed
  float* conv = nullptr;         // taps of a convolution: [cols][conv_C] from channel conv_at on, last column first
  int conv_C = 0, conv_at = 0;
  int64_t rows = 0, cols = 0;
};

bool find_target(Model* M, const std::string& n, Target* t) {
  const lmb200_model_config& c = M->cfg;
  auto vec = [&](float* d, int64_t len) { t->plain = d; t->vec = true; t->rows = 1; t->cols = len; return true; };
  auto mat = [&](void* d, const WMap& m, int slot) {
    t->tiled = d; t->map = &m; t->slot = slot; t->rows = m.src_rows[slot]; t->cols = m.src_cols[slot];
    return true;
  };
  if (n == "embed") {
    if (M->tied_head) mat(M->lm_head, M->m_head, 0);
    t->plain = M->embed; t->rows = c.vocab; t->cols = c.hidden;
    return true;
  }
  if (n == "final.norm") return vec(M->final_norm, c.hidden);
  if (n == "head" && !M->tied_head) return mat(M->lm_head, M->m_head, 0);
  if (n == "side.embed" && M->side_dim) { t->plain = M->side_embed; t->rows = c.vocab; t->cols = (int64_t)c.n_layers * M->side_dim; return true; }
  int layer = -1, used = 0;
  if (sscanf(n.c_str(), "l%d.%n", &layer, &used) < 1 || used == 0 || layer < 0 || layer >= c.n_layers) return false;
  const std::string tail = n.substr(used);
  LayerSpec& s = M->specs[layer];
  LayeredWeights& w = M->lw[layer];
  if (tail == "norm1") return vec(w.norm, c.hidden);
  const bool latent = is_latent(s);
  if (post_norm(M)) {
    if (s.c.ff && tail == "norm2") return vec(w.norm2, c.hidden);
    if (s.c.ff && tail == "mlp.gate") return mat(w.w_gu, s.m_gu, 0);
    if (s.c.ff && tail == "mlp.up") return mat(w.w_gu, s.m_gu, 1);
    if (s.c.ff && tail == "mlp.down") return mat(w.w_down, s.m_down, 0);
    if (M->side_dim && tail == "side.gate") return mat(w.w_sg, s.m_sg, 0);
    if (M->side_dim && tail == "side.proj") return mat(w.w_sp, s.m_sp, 0);
    if (M->side_dim && tail == "side.norm") return vec(w.side_norm, c.hidden);
    if (tail == "mix.o") return mat(w.w_out, s.m_out, 0);
    if (tail == "mix.q") return mat(w.w_in, s.m_in, 0);
    const bool own = !is_attention(s) || s.c.kv_from < 0;
    if (own && tail == "mix.k") return mat(w.w_in, s.m_in, 1);
    if (own && tail == "mix.v") return mat(w.w_in, s.m_in, 2);
    if (is_lightning(s)) {
      if (tail == "mix.g") return mat(w.w_in, s.m_in, R_G);
      if (tail == "mix.norm") return vec(w.mix_norm, out_width(s));
    }
    if (!is_delta(s)) return false;
    if (tail == "mix.b") return mat(w.w_in, s.m_in, D_B);
    if (tail == "mix.a1") return mat(w.w_in, s.m_in, D_A1);
    if (tail == "mix.g1") return mat(w.w_in, s.m_in, D_G1);
    if (tail == "mix.a2") return mat(w.w_lr, s.m_lr, 0);
    if (tail == "mix.g2") return mat(w.w_lr, s.m_lr, 1);
    if (tail == "mix.norm") return vec(w.mix_norm, s.c.vdim);
    if (tail == "mix.A_log") { t->offset = 0.f; return vec(w.a_log, s.c.heads); }
    if (tail == "mix.dt_bias") { t->offset = -2.f; return vec(w.dt_bias, (int64_t)s.c.heads * s.c.dim); }      // decays of about 0.9
    const int kd = s.c.kv_heads * s.c.dim;
    auto conv = [&](int at, int rows) { t->conv = w.conv; t->conv_C = delta_channels(s); t->conv_at = at; t->rows = rows; t->cols = s.c.conv; return true; };
    if (tail == "mix.q.conv") return conv(0, kd);
    if (tail == "mix.k.conv") return conv(kd, kd);
    if (tail == "mix.v.conv") return conv(2 * kd, out_width(s));
    return false;
  }
  if (s.c.ff && tail == "mlp.up") return mat(w.w_in, s.m_in, latent ? (int)L_UP : (int)R_UP);
  if (s.c.ff && tail == "mlp.down") return mat(w.w_out, s.m_out, 1);
  if (tail == "mix.o") return mat(w.w_out, s.m_out, 0);
  if (latent) {
    if (tail == "mix.dq") return mat(w.w_in, s.m_in, L_DQ);
    if (tail == "mix.dq.norm") return vec(w.q_norm, s.c.q_rank);
    if (tail == "mix.uq") return mat(w.w_uq, s.m_uq, 0);
    if (tail == "mix.g") return mat(w.w_in, s.m_in, L_G);
    if (s.c.kv_from < 0 && tail == "mix.dkv") return mat(w.w_in, s.m_in, L_DKV);
    if (s.c.kv_from < 0 && tail == "mix.dkv.norm") return vec(w.kv_norm, s.c.kv_rank);
    if (tail == "mix.uk") { mat(w.w_ukv, s.m_ukv, 0); t->plain = w.w_ukt; t->head = s.c.dim; return true; }
    if (tail == "mix.uv") { mat(w.w_ukv, s.m_ukv, 1); t->plain = w.w_uv; return true; }
    return false;
  }
  if (tail == "mix.q") return mat(w.w_in, s.m_in, R_Q);
  if (tail == "mix.k") return mat(w.w_in, s.m_in, R_K);
  if (tail == "mix.v") return mat(w.w_in, s.m_in, R_V);
  if (tail == "mix.g") return mat(w.w_in, s.m_in, R_G);
  return false;
}

__global__ void fill_conv_kernel(float* __restrict__ conv, int C, int at, int rows, int taps, const float* __restrict__ src, int colmajor, uint64_t key,
                                 float scale) {
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < rows * taps; i += gridDim.x * blockDim.x) {
    const int c = i / taps, j = i - c * taps;
    conv[(int64_t)(taps - 1 - j) * C + at + c] = src ? src[colmajor ? c + rows * j : i] : synth_value(key, (uint64_t)i, scale, 0.f);
  }
}

// fills a tensor from `src` (device float32) or, src == NULL, from the generator
int32_t fill_target(Model* M, const Target& t, uint64_t key, const float* src, int layout, float scale) {
  if (t.conv) {                      // generated taps are of order one, as a trained convolution's are
    fill_conv_kernel<<<64, 256, 0, M->ctx->stream>>>(t.conv, t.conv_C, t.conv_at, (int)t.rows, (int)t.cols, src, layout, key, 0.5f / 131072.0f);
    M->ctx->launches++;
    LMB_CUDA(cudaGetLastError());
    return LMB200_OK;
  }
  if (t.vec) return fill_plain_dt(M, LMB200_F32, t.plain, t.rows, t.cols, key, src, 0, scale, src ? 0.f : t.offset);
  if (t.plain) LMB_TRY(fill_plain_dt(M, M->cfg.dtype, t.plain, t.rows, t.cols, key, src, layout, scale, 0.f, t.head));
  if (!t.tiled) return LMB200_OK;
  FillSrc f{};
  f.only_slot = t.slot; f.colmajor = layout; f.scale = scale;
  f.key[t.slot] = key; f.src[t.slot] = src;
  return fill_tiled_dt(M, t.tiled, *t.map, f);
}

}  // namespace

void layered_free_model(Model* M) {
  for (LayeredWeights& w : M->lw) {
    cudaFree(w.w_in); cudaFree(w.w_out); cudaFree(w.w_uq); cudaFree(w.w_ukv); cudaFree(w.w_ukt); cudaFree(w.w_uv);
    cudaFree(w.w_gu); cudaFree(w.w_down); cudaFree(w.w_sg); cudaFree(w.w_sp); cudaFree(w.w_lr); cudaFree(w.norm2); cudaFree(w.side_norm);
    cudaFree(w.mix_norm); cudaFree(w.conv); cudaFree(w.a_log); cudaFree(w.dt_bias);
    cudaFree(w.norm); cudaFree(w.q_norm); cudaFree(w.kv_norm); cudaFree(w.inv_freq); cudaFree(w.decay);
  }
  M->lw.clear();
  cudaFree(M->side_embed);
  M->side_embed = nullptr;
}

bool layered_has_state(const Model* M) {
  for (const LayerSpec& s : M->specs)
    if (has_state(s)) return true;
  return false;
}

std::vector<std::string> layered_weight_names(const Model* M) {
  std::vector<std::string> v = {"embed", "final.norm"};
  if (!M->tied_head) v.push_back("head");
  if (M->side_dim) v.push_back("side.embed");
  for (int l = 0; l < M->cfg.n_layers; ++l) {
    const LayerSpec& s = M->specs[l];
    const std::string p = "l" + std::to_string(l) + ".";
    v.push_back(p + "norm1");
    std::vector<const char*> mix = {"q", "k", "v", "g", "o"};
    if (is_latent(s)) {
      mix = {"dq", "dq.norm", "uq", "uk", "uv", "g", "o"};
      if (s.c.kv_from < 0) { mix.push_back("dkv"); mix.push_back("dkv.norm"); }
    } else if (is_attention(s)) {
      mix = {"q", "o"};
      if (s.c.kv_from < 0) { mix.push_back("k"); mix.push_back("v"); }
    } else if (is_delta(s)) {
      mix = {"q", "q.conv", "k", "k.conv", "v", "v.conv", "b", "A_log", "dt_bias", "a1", "a2", "g1", "g2", "norm", "o"};
    } else if (is_lightning(s)) {
      mix.push_back("norm");
    }
    for (const char* t : mix) v.push_back(p + "mix." + t);
    if (s.c.ff) { v.push_back(p + "mlp.up"); v.push_back(p + "mlp.down"); }
    if (s.c.ff && post_norm(M)) { v.push_back(p + "mlp.gate"); v.push_back(p + "norm2"); }
    if (M->side_dim)
      for (const char* t : {"gate", "proj", "norm"}) v.push_back(p + "side." + t);
  }
  return v;
}

int32_t layered_set_weight(Model* M, const char* name, const float* host, int32_t rank, const int64_t* dims, int32_t layout) {
  Ctx* ctx = M->ctx;
  Target t;
  if (!find_target(M, name, &t)) return fail(LMB200_ENOTFOUND, "set_weight: unknown tensor '%s'", name);
  LMB_TRY(check_weight_shape(name, rank, dims, t.rows, t.cols));
  float* stage = nullptr;
  LMB_TRY(dmalloc((void**)&stage, t.rows * t.cols * 4, false, ctx->stream));
  int32_t rc = LMB200_OK;
  if (cudaMemcpyAsync(stage, host, (size_t)(t.rows * t.cols) * 4, cudaMemcpyHostToDevice, ctx->stream) != cudaSuccess)
    rc = fail(LMB200_ECUDA, "set_weight: upload failed");
  if (rc == LMB200_OK) rc = fill_target(M, t, 0, stage, layout, 0.f);
  cudaStreamSynchronize(ctx->stream);
  cudaFree(stage);
  if (rc == LMB200_OK) M->weights_set.insert(name);
  return rc;
}

int32_t layered_init_random(Model* M, uint64_t seed, float sigma) {
  Ctx* ctx = M->ctx;
  LMB_CUDA(cudaSetDevice(ctx->device));
  uint64_t id = kIdLayered;
  for (const std::string& n : layered_weight_names(M)) {
    Target t;
    if (!find_target(M, n, &t)) return fail(LMB200_EINVAL, "init_random: '%s'", n.c_str());
    LMB_TRY(fill_target(M, t, stream_key(seed, id++), nullptr, LMB200_ROWMAJOR, sigma / 131072.0f));
  }
  LMB_CUDA(cudaStreamSynchronize(ctx->stream));
  M->all_weights_set = true;
  return LMB200_OK;
}

// ---------------------------------------------------------------------------------------------
// session
// ---------------------------------------------------------------------------------------------
namespace {

template <typename F>
int64_t max_over(const Model* M, F f) {
  int64_t m = 0;
  for (const LayerSpec& s : M->specs) m = std::max<int64_t>(m, f(s));
  return m;
}

void free_rows(RowsBuf& r) {
  cudaFree(r.base);
  r = RowsBuf();
}

// the buffers for T tokens, carved out of one allocation (a larger request replaces it)
int32_t ensure_rows(Session* S, RowsBuf& r, int64_t T, int64_t n_want) {
  const Model* M = S->m;
  const int64_t e = M->esz, W = M->cfg.hidden;
  const int64_t need_meta = 4 * T + 3 * S->B + n_want;
  if (T <= r.cap_T && need_meta <= 4 * r.cap_T + 3 * S->B + r.cap_T) return LMB200_OK;
  T = std::max<int64_t>(T, r.cap_T);
  free_rows(r);
  const int64_t blk = std::min<int64_t>(T, kBlockTokens);
  r.max_half = (int)max_over(M, [](const LayerSpec& s) { return s.c.rot_dims / 2; });
  struct Piece { void** p; int64_t bytes; };
  const Piece pieces[] = {
      {(void**)&r.x, T * W * 4},
      {(void**)&r.delta, T * W * 4},
      {&r.xn, T * row_ld((int)W) * e},
      {(void**)&r.proj, T * max_over(M, [&](const LayerSpec& s) { return std::max<int64_t>(is_latent(s) ? (int64_t)s.n_store * 4 : (int64_t)s.n_store * e, e == 4 ? s.m_gu.rows * e : 0); })},
      {&r.xq, T * row_ld((int)max_over(M, [](const LayerSpec& s) { return s.c.q_rank; })) * e},
      {&r.q, T * max_over(M, [](const LayerSpec& s) { return is_latent(s) ? q_width(s) : is_attention(s) ? s.c.heads * s.c.dim : is_delta(s) ? row_ld(delta_channels(s)) : 0; }) * e},
      {&r.qa, blk * max_over(M, [](const LayerSpec& s) { return is_latent(s) ? (int64_t)s.c.heads * s.lat_ld : 0; }) * e},
      {&r.cat, T * max_over(M, [](const LayerSpec& s) { return row_ld(s.m_out.K); }) * e},
      {&r.packed, T * max_over(M, [](const LayerSpec& s) { return is_latent(s) ? s.lat_ld : 0; }) * e},
      {&r.act, T * max_over(M, [&](const LayerSpec& s) { return post_norm(M) ? row_ld(s.c.ff) : 0; }) * e},
      {&r.side, T * row_ld(M->side_dim) * e},
      {&r.lr_in, T * max_over(M, [](const LayerSpec& s) { return is_delta(s) ? row_ld(s.m_lr.K) : 0; }) * e},
      {&r.gate, T * max_over(M, [](const LayerSpec& s) { return is_delta(s) ? row_ld(out_width(s)) : 0; }) * e},
      {(void**)&r.beta, T * max_over(M, [](const LayerSpec& s) { return is_delta(s) ? s.c.heads : 0; }) * 4},
      {(void**)&r.log_g, T * max_over(M, [](const LayerSpec& s) { return is_delta(s) ? (int64_t)s.c.heads * s.c.dim : 0; }) * 4},
      {(void**)&r.rq, T * max_over(M, [](const LayerSpec& s) { return is_delta(s) ? s.c.kv_heads : 0; }) * 4},
      {(void**)&r.rk, T * max_over(M, [](const LayerSpec& s) { return is_delta(s) ? s.c.kv_heads : 0; }) * 4},
      {(void**)&r.ssq, T * max_over(M, [](const LayerSpec& s) { return is_lightning(s) ? s.c.heads : 0; }) * 4},
      {(void**)&r.angles, M->cfg.dtype == LMB200_BF16 ? (int64_t)M->rot_freqs.size() * T * r.max_half * 8 : 0},
      {(void**)&r.meta, (5 * T + 3 * S->B) * 4},
  };
  int64_t total = 0;
  for (const Piece& p : pieces) total += round_up(p.bytes, 256);
  LMB_TRY(dmalloc(&r.base, total, true, M->ctx->stream));
  char* at = reinterpret_cast<char*>(r.base);
  for (const Piece& p : pieces) { *p.p = at; at += round_up(p.bytes, 256); }
  r.bytes = total;
  r.cap_T = T;
  return LMB200_OK;
}

// four consecutive elements in one store
__device__ __forceinline__ void store4(float* o, float a, float b, float c, float d) { *reinterpret_cast<float4*>(o) = make_float4(a, b, c, d); }
__device__ __forceinline__ void store4(__nv_bfloat16* o, float a, float b, float c, float d) {
  reinterpret_cast<__nv_bfloat162*>(o)[0] = __floats2bfloat162_rn(a, b);
  reinterpret_cast<__nv_bfloat162*>(o)[1] = __floats2bfloat162_rn(c, d);
}

// x[t] <- embedding row (tokens given) or x[t] + delta[t]; xn[t] = RMSNorm(x[t]) w in the model dtype.  Rows in order, or the rows
// `pick` chooses (then x itself is left alone).  capture [.., n]: the new row of every sequence's last token.
template <typename WT>
__global__ void __launch_bounds__(256) rows_norm_kernel(float* __restrict__ x, const float* __restrict__ delta, const int* __restrict__ tokens,
                                                        const WT* __restrict__ embed, int vocab, const int* __restrict__ pick,
                                                        const float* __restrict__ w, WT* __restrict__ xn, int ldn, int n, float eps,
                                                        float* __restrict__ capture, const int* __restrict__ last) {
  extern __shared__ __align__(16) float row[];
  __shared__ float red[8];
  pdl_launch_dependents();
  pdl_wait();
  const int i0 = blockIdx.x, tid = threadIdx.x;
  const int64_t t = pick ? pick[i0] : i0;
  const int tok = tokens ? tokens[t] : 0;
  const bool ok = tok >= 0 && tok < vocab;
  const int cap = capture && !pick ? last[t] : -1;
  float ss = 0.f;
  // whole vectors where the rows allow it (residual rows: the embedding and the captured rows take the other loop)
  if (!tokens && cap < 0 && (n & 3) == 0 && (ldn & 3) == 0) {
    float4* x4 = reinterpret_cast<float4*>(x + t * n);
    const float4* d4 = delta ? reinterpret_cast<const float4*>(delta + t * n) : nullptr;
    float4* r4 = reinterpret_cast<float4*>(row);
#pragma unroll 4
    for (int i = tid; i < (n >> 2); i += 256) {
      float4 v = x4[i];
      if (d4) { const float4 d = d4[i]; v.x += d.x; v.y += d.y; v.z += d.z; v.w += d.w; }
      if (!pick) x4[i] = v;
      r4[i] = v;
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int i = tid; i < n; i += 256) {
      float v;
      if (tokens) v = ok ? to_f32(embed[(int64_t)tok * n + i]) : 0.f;
      else v = x[t * n + i] + (delta ? delta[t * n + i] : 0.f);
      if (!pick) x[t * n + i] = v;
      if (cap >= 0) capture[(int64_t)cap * n + i] = v;
      row[i] = v;
      ss += v * v;
    }
  }
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) tot += red[i];
  const float inv = 1.0f / sqrtf(tot / (float)n + eps);
  if (!xn) return;
  if ((n & 3) == 0 && (ldn & 3) == 0) {
    const float4* r4 = reinterpret_cast<const float4*>(row);
    const float4* w4 = reinterpret_cast<const float4*>(w);
    for (int i = tid; i < (n >> 2); i += 256) {
      const float4 v = r4[i], g = w4[i];
      store4(xn + (int64_t)i0 * ldn + 4 * i, v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w);
    }
    return;
  }
  for (int i = tid; i < n; i += 256) xn[(int64_t)i0 * ldn + i] = from_f32<WT>(row[i] * inv * w[i]);
}

// x[t] <- scale * embedding row (tokens given) or x[t] + rms(inv y[t]) w, rms(z) = z / sqrt(mean z^2 + eps); xn[t] = x[t] in the model
// dtype.  inv: 1, or (ssq given, heads sums per row) 1 / sqrt(sum / ssq_n + eps).  capture as in rows_norm_kernel.
template <typename WT>
__global__ void __launch_bounds__(256) rows_post_kernel(float* __restrict__ x, const float* __restrict__ y, const int* __restrict__ tokens,
                                                        const WT* __restrict__ embed, int vocab, float scale, const float* __restrict__ w,
                                                        const float* __restrict__ ssq, int heads, int ssq_n, WT* __restrict__ xn, int ldn, int n,
                                                        float eps, float* __restrict__ capture, const int* __restrict__ last) {
  extern __shared__ __align__(16) float row[];
  __shared__ float red[8];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x;
  const int64_t t = blockIdx.x;
  if (tokens) {
    const int tok = tokens[t];
    const bool ok = tok >= 0 && tok < vocab;
    for (int i = tid; i < n; i += 256) {
      const float v = ok ? to_f32(embed[(int64_t)tok * n + i]) * scale : 0.f;
      x[t * n + i] = v;
      xn[t * ldn + i] = from_f32<WT>(v);
    }
    return;
  }
  float inv = 1.f;
  if (ssq) {
    float s = 0.f;
    for (int i = 0; i < heads; ++i) s += ssq[t * heads + i];
    inv = 1.0f / sqrtf(s / (float)ssq_n + eps);
  }
  const int cap = capture ? last[t] : -1;
  const bool vec = cap < 0 && (n & 3) == 0 && (ldn & 3) == 0;
  float ss = 0.f;
  if (vec) {
    const float4* y4 = reinterpret_cast<const float4*>(y + t * n);
    float4* r4 = reinterpret_cast<float4*>(row);
#pragma unroll 4
    for (int i = tid; i < (n >> 2); i += 256) {
      float4 v = y4[i];
      v.x *= inv; v.y *= inv; v.z *= inv; v.w *= inv;
      r4[i] = v;
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int i = tid; i < n; i += 256) {
      const float v = y[t * n + i] * inv;
      row[i] = v;
      ss += v * v;
    }
  }
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) tot += red[i];
  const float f = 1.0f / sqrtf(tot / (float)n + eps);
  if (vec) {
    float4* x4 = reinterpret_cast<float4*>(x + t * n);
    const float4* r4 = reinterpret_cast<const float4*>(row);
    const float4* w4 = reinterpret_cast<const float4*>(w);
#pragma unroll 4
    for (int i = tid; i < (n >> 2); i += 256) {
      float4 v = x4[i];
      const float4 r = r4[i], g = w4[i];
      v.x += r.x * f * g.x; v.y += r.y * f * g.y; v.z += r.z * f * g.z; v.w += r.w * f * g.w;
      x4[i] = v;
      store4(xn + t * ldn + 4 * i, v.x, v.y, v.z, v.w);
    }
    return;
  }
  for (int i = tid; i < n; i += 256) {
    const float v = x[t * n + i] + row[i] * f * w[i];
    x[t * n + i] = v;
    if (cap >= 0) capture[(int64_t)cap * n + i] = v;
    xn[t * ldn + i] = from_f32<WT>(v);
  }
}

// float32 feed-forward: the stacked projection's rows (8 gate, 8 up) to act[t, i] = silu(gate_i) up_i
__global__ void __launch_bounds__(256) silu_gate_rows_kernel(const float* __restrict__ gu, int ldg, float* __restrict__ act, int lda, int ff, int T) {
  pdl_launch_dependents();
  pdl_wait();
  for (int64_t o = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; o < (int64_t)T * ff; o += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = o / ff;
    const int i = (int)(o - t * ff);
    const float* r = gu + t * ldg + (i >> 3) * 16 + (i & 7);
    act[t * lda + i] = silu_f32(r[0]) * r[8];
  }
}

// float32 GEMM over many tokens on the CUDA cores: 64 rows x 64 tokens per CTA, W in the 16 x 32 tiles of the float32 layout
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ W, const float* __restrict__ X, int ldx, int T, int rows, int K,
                                                       const RowSegs segs) {
  __shared__ float ws[32][68], xs[32][68];              // [k][row], [k][token]
  pdl_launch_dependents();
  pdl_wait();
  const int row0 = blockIdx.x * 64, t0 = blockIdx.y * 64, tid = threadIdx.x;
  const int KC = (K + 31) >> 5, RB = (rows + 15) >> 4;
  const int tr = (tid & 15) * 4, tt = (tid >> 4) * 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int kc = 0; kc < KC; ++kc) {
    for (int i = tid; i < 64 * 32; i += 256) {
      const int r = i >> 5, k = i & 31;
      ws[k][r] = ((row0 + r) >> 4) < RB ? W[wtile_offset(row0 + r, kc * 32 + k, KC)] : 0.f;
      xs[k][r] = t0 + r < T && kc * 32 + k < K ? X[(int64_t)(t0 + r) * ldx + kc * 32 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 32; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&ws[k][tr]), b = *reinterpret_cast<const float4*>(&xs[k][tt]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
  for (int i = 0; i < 4; ++i) {
    const int row = row0 + tr + i;
    for (int s = 0; s < segs.n; ++s) {
      const RowSeg sg = segs.s[s];
      const int r = row - sg.row0;
      if (r < 0 || r >= sg.rows) continue;
      for (int j = 0; j < 4; ++j) {
        if (t0 + tt + j >= T) continue;
        float y = acc[i][j];
        if (sg.kind == SEG_RELU2) { y = fmaxf(y, 0.f); y = y * y; }
        else if (sg.kind == SEG_SILU) y = y / (1.0f + expf(-y));
        else if (sg.kind == SEG_SOFTCAP && segs.softcap > 0.f) y = segs.softcap * tanhf(y / segs.softcap);
        else if (sg.kind == SEG_SIGMOID) y = sigmoid_f32(y);
        else if (sg.kind == SEG_DECAY) y = log_decay_f32(y, sg.rate[r / sg.head], sg.bias[r]);
        else if (sg.kind == SEG_GELU_TOKEN) {
          const int tok = sg.tokens[t0 + tt + j];
          y = tok >= 0 && tok < sg.table_rows ? gelu_tanh_f32(y) * reinterpret_cast<const float*>(sg.table)[(int64_t)tok * sg.table_pitch + r] : 0.f;
        }
        reinterpret_cast<float*>(sg.dst)[(int64_t)(t0 + tt + j) * sg.pitch + r] = y;
      }
    }
  }
}

int32_t rows_gemm(const Model* M, const void* W, const WMap& m, const void* X, int ldx, int T, const RowSegs& segs, cudaStream_t st) {
  Ctx* ctx = M->ctx;
  if (M->cfg.dtype == LMB200_BF16) return gemm_segments_bf16(ctx, W, X, ldx, T, m.rows, m.K, segs, st);
  LMB_REQUIRE(ceil_div(T, 64) <= 65535, "layered: %d tokens in one call", T);
  LMB_CUDA(launch_k(gemm_f32_kernel, dim3((unsigned)ceil_div(m.rows, 64), (unsigned)ceil_div(T, 64)), dim3(256), 0, st, (const float*)W,
                    (const float*)X, ldx, T, m.rows, m.K, segs));
  ctx->launches++;
  return LMB200_OK;
}

LatentView latent_view(const Session* S, int l) {
  const Model* M = S->m;
  const LayerSpec& s = M->specs[l];
  LatentView v;
  v.H = s.c.heads; v.dim = s.c.dim; v.vdim = s.c.vdim; v.q_rank = s.c.q_rank; v.kv_rank = s.c.kv_rank;
  v.rot_dim = s.c.rot_dim; v.rot_dims = s.c.rot_dims; v.rot_interleaved = s.c.rot_layout == LMB200_ROT_INTERLEAVED;
  v.rot = s.lat_rot; v.ld = s.lat_ld;
  v.seq_stride = (int64_t)S->cap * s.lat_ld;
  v.inv_freq = M->lw[l].inv_freq;
  v.scale = s.c.scale; v.eps = M->cfg.rms_eps;
  return v;
}

RetentionView retention_view(const Session* S, int l) {
  const Model* M = S->m;
  const LayerSpec& s = M->specs[l];
  RetentionView v;
  v.B = S->B;
  v.H = s.c.heads; v.dim = s.c.dim; v.vdim = s.c.vdim; v.rot_dims = s.c.rot_dims;
  v.inv_freq = M->lw[l].inv_freq; v.decay = M->lw[l].decay; v.decay_pitch = kDecayPow;
  v.eps = M->cfg.rms_eps;
  v.state = S->state[l];
  v.k_scale = is_lightning(s) ? 1.0f : 1.0f / sqrtf((float)s.c.dim);
  v.out_w = is_lightning(s) ? M->lw[l].mix_norm : nullptr;
  return v;
}

WindowView window_view(const Session* S, int l) {
  const Model* M = S->m;
  const LayerSpec& s = M->specs[l];
  const int src = cache_layer(M, l);
  WindowView v;
  v.H = s.c.heads; v.G = s.c.kv_heads; v.dim = s.c.dim; v.vdim = s.c.vdim;
  v.k_ld = s.k_ld; v.v_ld = s.v_ld; v.cap = S->cap;
  v.keys = S->keys[src]; v.values = S->values[src];
  v.rot_dims = s.c.rot_dims; v.rot_interleaved = s.c.rot_layout == LMB200_ROT_INTERLEAVED;
  v.inv_freq = M->lw[l].inv_freq; v.rot_scale = rotation_scale(s.c);
  v.scale = s.c.scale; v.score_cap = s.c.score_cap; v.eps = M->cfg.rms_eps; v.window = s.c.window;
  return v;
}

DeltaView delta_view(const Session* S, int l) {
  const Model* M = S->m;
  const LayerSpec& s = M->specs[l];
  const LayeredWeights& w = M->lw[l];
  DeltaView v;
  v.B = S->B; v.H = s.c.heads; v.G = s.c.kv_heads; v.dim = s.c.dim; v.vdim = s.c.vdim; v.taps = s.c.conv;
  v.eps = M->cfg.rms_eps;
  v.state = S->state[l]; v.ring = S->conv[l];
  v.conv = w.conv; v.a_log = w.a_log; v.dt_bias = w.dt_bias; v.norm = w.mix_norm;
  return v;
}

// What a rows step runs over: packed tokens and, on the host, how they divide into sequences (empty: one token per sequence)
struct RowsRun {
  int T = 0;
  const int *tokens = nullptr, *seq = nullptr, *pos = nullptr, *last = nullptr, *start = nullptr, *len = nullptr, *pos0 = nullptr;
  int max_len = 1;
  int ctx_len = 0;                       // no token looks at more positions than this
  std::vector<int> h_start, h_len, h_pos0;
};

template <typename WT>
int32_t norm_rows(Session* S, RowsBuf& r, const RowsRun& run, int n_rows, const float* delta, bool embed, const int* pick, const float* w, void* xn,
                  float* capture, cudaStream_t st) {
  const Model* M = S->m;
  const int W = M->cfg.hidden;
  LMB_CUDA(launch_k(rows_norm_kernel<WT>, dim3((unsigned)n_rows), dim3(256), (size_t)W * 4, st, r.x, delta, embed ? run.tokens : (const int*)nullptr,
                    (const WT*)M->embed, M->cfg.vocab, pick, w, (WT*)xn, row_ld(W), W, M->cfg.rms_eps, capture, run.last));
  M->ctx->launches++;
  return LMB200_OK;
}

// The angles of this step's tokens (bf16 models), computed once for all layers with the same frequencies.
int32_t step_angles(Session* S, RowsBuf& r, const RowsRun& run, int l, float2** tab, cudaStream_t st) {
  Model* M = S->m;
  const int id = M->lw[l].rot_id, n = M->specs[l].c.rot_dims / 2;
  *tab = r.angles + (int64_t)id * r.cap_T * r.max_half;
  if (!r.angles_valid[id]) {
    LMB_TRY(angle_table(M->ctx, *tab, M->lw[l].inv_freq, n, run.pos, run.T, st));
    r.angles_valid[id] = true;
  }
  return LMB200_OK;
}

// Makes `sg` a SEG_ROT segment of layer l: heads of `head` rows whose features from `off` on rotate.
int32_t rotate_segment(Session* S, RowsBuf& r, const RowsRun& run, int l, RowSeg& sg, int head, int off, cudaStream_t st) {
  const int n = S->m->specs[l].c.rot_dims / 2;
  float2* tab = nullptr;
  LMB_TRY(step_angles(S, r, run, l, &tab, st));
  sg.rot = tab; sg.rot_head = head; sg.rot_off = off; sg.rot_dims = 2 * n;
  return LMB200_OK;
}

// scratch of the absorbed attention in a rows step
int32_t ensure_attn_scratch(Session* S, const LatentAttnPlan& plan) {
  LayeredScratch& Z = *S->lay;
  cudaStream_t st = S->m->ctx->stream;
  if (plan.part_floats > Z.prompt_part_floats) {
    cudaFree(Z.prompt_part);
    Z.prompt_part = nullptr; Z.prompt_part_floats = 0;
    LMB_TRY(dmalloc((void**)&Z.prompt_part, plan.part_floats * 4, false, st));
    Z.prompt_part_floats = plan.part_floats;
  }
  return LMB200_OK;
}

int32_t latent_rows(Session* S, RowsBuf& r, const RowsRun& run, int l, bool graph, cudaStream_t st) {
  Model* M = S->m;
  Ctx* ctx = M->ctx;
  const LayerSpec& s = M->specs[l];
  LayeredWeights& w = M->lw[l];
  LayeredScratch& Z = *S->lay;
  const int dt = M->cfg.dtype, T = run.T, e = M->esz, ldc = row_ld(s.m_out.K), ldq = row_ld(s.c.q_rank);
  const bool own = s.c.kv_from < 0;
  RowSegs in;
  in.add(s.row0[L_DQ], s.c.q_rank, SEG_F32, r.proj + s.row0[L_DQ], s.n_store);
  if (own) in.add(s.row0[L_DKV], s.c.kv_rank + s.c.rot_dim, SEG_F32, r.proj + s.row0[L_DKV], s.n_store);
  in.add(s.row0[L_G], s.c.heads, SEG_F32, r.proj + s.row0[L_G], s.n_store);
  if (s.c.ff) in.add(s.row0[L_UP], s.c.ff, SEG_RELU2, (char*)r.cat + (int64_t)s.cat0 * e, ldc);
  LMB_TRY(rows_gemm(M, w.w_in, s.m_in, r.xn, row_ld(M->cfg.hidden), T, in, st));
  LatentView v = latent_view(S, l);
  v.T = T; v.seq = run.seq; v.pos = run.pos;
  void* cache = S->latent[cache_layer(M, l)];
  LMB_TRY(latent_prep(ctx, dt, v, r.proj, s.n_store, s.row0[L_DQ], own ? s.row0[L_DKV] : 0, w.q_norm, w.kv_norm, r.xq, ldq, 0,
                      own ? cache : nullptr, own ? r.packed : nullptr, st));
  if (own) r.packed_layer = l;
  RowSegs qs;
  const bool rot = dt == LMB200_BF16 && s.c.rot_dims > 0 && v.rot_interleaved && s.c.dim % 2 == 0 && s.c.rot_dim % 2 == 0;
  qs.add(0, q_width(s), rot ? SEG_ROT : SEG_ACT, r.q, q_width(s));
  if (rot) {
    LMB_TRY(rotate_segment(S, r, run, l, qs.s[0], s.c.dim + s.c.rot_dim, s.c.dim, st));
    v.q_rotated = 1;
  }
  LMB_TRY(rows_gemm(M, w.w_uq, s.m_uq, r.xq, ldq, T, qs, st));
  const float* gate = r.proj + s.row0[L_G];
  auto absorbed = [&](int t0, int t1) -> int32_t {
    for (; t0 < t1; t0 += kBlockTokens) {
      LatentView b = v;
      b.T = std::min(kBlockTokens, t1 - t0); b.seq = run.seq + t0; b.pos = run.pos + t0;
      LMB_TRY(latent_absorb(ctx, dt, b, (const char*)r.q + (int64_t)t0 * q_width(s) * e, 0, w.w_ukt, r.qa, st));
      const LatentAttnPlan plan = graph ? Z.attn[l] : latent_attn_plan(ctx, dt, b, b.T, run.ctx_len);
      if (!graph) LMB_TRY(ensure_attn_scratch(S, plan));
      float* part = graph ? Z.attn_part : Z.prompt_part;
      LMB_TRY(latent_attend(ctx, dt, b, r.qa, cache, plan, part, st));
      LMB_TRY(latent_expand(ctx, dt, b, part, plan, w.w_uv, gate + (int64_t)t0 * s.n_store, s.n_store, (char*)r.cat + (int64_t)t0 * ldc * e, ldc, 0, st));
    }
    return LMB200_OK;
  };
  const bool flash = dt == LMB200_BF16 && !graph && flash_tc_split_supported(s.c.dim, s.c.rot_dim, s.c.vdim);
  // keys and values of `rows` latent rows, then the attention of n queries per sequence over them
  auto expanded = [&](int t0, const void* lat, int64_t rows, int n_batch, int n, int64_t ctx_rows) -> int32_t {
    const int64_t kw = (int64_t)s.c.heads * s.c.dim, vw = out_width(s);
    const int64_t bytes = round_up(rows * kw * 2, 256) + rows * vw * 2;
    if (bytes > Z.expanded_bytes) {
      LMB_CUDA(cudaStreamSynchronize(st));
      cudaFree(Z.expanded);
      Z.expanded = nullptr; Z.expanded_bytes = 0;
      LMB_TRY(dmalloc(&Z.expanded, bytes, false, st));
      Z.expanded_bytes = bytes;
    }
    void* kx = Z.expanded;
    void* vx = (char*)Z.expanded + round_up(rows * kw * 2, 256);
    RowSegs kv;
    kv.add(s.m_ukv.row_off[0], (int)kw, SEG_ACT, kx, (int)kw);
    kv.add(s.m_ukv.row_off[1], (int)vw, SEG_ACT, vx, (int)vw);
    LMB_TRY(rows_gemm(M, w.w_ukv, s.m_ukv, lat, s.lat_ld, (int)rows, kv, st));
    FlashSplitView f;
    f.H = s.c.heads; f.dn = s.c.dim; f.dr = s.c.rot_dim; f.dv = s.c.vdim;
    f.q_s = q_width(s); f.q_h = s.c.dim + s.c.rot_dim; f.q_b = (int64_t)n * f.q_s;
    f.o_s = ldc; f.o_h = s.c.vdim; f.o_b = (int64_t)n * ldc;
    f.k_s = kw; f.k_h = s.c.dim; f.k_b = ctx_rows * kw;
    f.v_s = vw; f.v_h = s.c.vdim; f.v_b = ctx_rows * vw;
    f.kr_s = s.lat_ld; f.kr_b = ctx_rows * s.lat_ld;
    f.gate = gate + (int64_t)t0 * s.n_store; f.gate_pitch = s.n_store;
    return flash_tc_launch_split(ctx, (char*)r.cat + (int64_t)t0 * ldc * e, (const char*)r.q + (int64_t)t0 * q_width(s) * e, kx,
                                 (const char*)lat + (int64_t)s.lat_rot * e, vx, f, n_batch, n, ctx_rows, s.c.scale, st);
  };
  auto rotate = [&](int t0, int n) -> int32_t {
    if (rot) return LMB200_OK;
    LatentView b = v;
    b.T = n; b.pos = run.pos + t0;
    return latent_rotate_q(ctx, b, (char*)r.q + (int64_t)t0 * q_width(s) * e, st);
  };
  if (!flash) return absorbed(0, T);
  bool uniform = S->B > 1 && r.packed_layer == cache_layer(M, l);
  for (int b = 0; b < S->B; ++b) uniform = uniform && run.h_pos0[b] == 0 && run.h_len[b] == run.h_len[0];
  if (uniform && run.h_len[0] >= kFlashMin && (int64_t)S->B * s.c.heads <= 65535) {       // fresh prompts of one length: all at once
    LMB_TRY(rotate(0, T));
    return expanded(0, r.packed, T, S->B, run.h_len[0], run.h_len[0]);
  }
  int pending = 0;                                      // first token of the run of short portions not yet attended
  for (int b = 0; b < S->B; ++b) {
    const int t0 = run.h_start[b], n = run.h_len[b];
    if (n < kFlashMin) continue;
    LMB_TRY(absorbed(pending, t0));
    pending = t0 + n;
    LMB_TRY(rotate(t0, n));
    const char* lat = (const char*)cache + (int64_t)b * S->cap * s.lat_ld * e;
    LMB_TRY(expanded(t0, lat, run.h_pos0[b] + n, 1, n, run.h_pos0[b] + n));
  }
  return absorbed(pending, T);
}

int32_t attention_rows(Session* S, RowsBuf& r, const RowsRun& run, int l, bool graph, cudaStream_t st) {
  Model* M = S->m;
  Ctx* ctx = M->ctx;
  const LayerSpec& s = M->specs[l];
  LayeredScratch& Z = *S->lay;
  const int dt = M->cfg.dtype, T = run.T, e = M->esz, ldc = row_ld(s.m_out.K), qw = s.c.heads * s.c.dim;
  const bool own = s.c.kv_from < 0;
  char* proj = reinterpret_cast<char*>(r.proj);
  RowSegs in;
  in.add(s.row0[D_Q], qw, SEG_ACT, r.q, qw);
  if (own) {
    in.add(s.row0[D_K], s.c.kv_heads * s.c.dim, SEG_ACT, proj + (int64_t)s.row0[D_K] * e, s.n_store);
    in.add(s.row0[D_V], s.c.kv_heads * s.c.vdim, SEG_ACT, proj + (int64_t)s.row0[D_V] * e, s.n_store);
  }
  LMB_TRY(rows_gemm(M, M->lw[l].w_in, s.m_in, r.xn, row_ld(M->cfg.hidden), T, in, st));
  WindowView v = window_view(S, l);
  v.T = T; v.seq = run.seq; v.pos = run.pos;
  if (dt == LMB200_BF16 && s.c.rot_dims > 0) {
    float2* tab = nullptr;
    LMB_TRY(step_angles(S, r, run, l, &tab, st));
    v.angles = tab;
  }
  WindowRows w;
  w.q = r.q; w.q_pitch = qw; w.in_f32 = dt != LMB200_BF16;
  if (own) {
    w.k = proj + (int64_t)s.row0[D_K] * e; w.v = proj + (int64_t)s.row0[D_V] * e;
    w.k_pitch = w.v_pitch = s.n_store;
  }
  LMB_TRY(window_prep(ctx, dt, v, w, r.q, st));
  WindowRows q;
  q.q_pitch = qw; q.in_f32 = 0;
  auto split = [&](int t0, int t1) -> int32_t {             // a few queries each: the cache is read once per token
    for (; t0 < t1; t0 += kBlockTokens) {
      WindowView b = v;
      b.T = std::min(kBlockTokens, t1 - t0); b.seq = run.seq + t0; b.pos = run.pos + t0;
      b.angles = nullptr;
      q.q = (const char*)r.q + (int64_t)t0 * qw * e;
      void* out = (char*)r.cat + (int64_t)t0 * ldc * e;
      if (graph) { LMB_TRY(window_attend(ctx, dt, b, q, Z.win[l], Z.attn_part, Z.win_cnt, out, ldc, 0, st)); continue; }
      const WindowPlan plan = window_plan(ctx, dt, b, b.T, run.ctx_len);
      LatentAttnPlan lp;
      lp.part_floats = plan.part_floats;
      LMB_TRY(ensure_attn_scratch(S, lp));
      if (plan.n_counters > Z.prompt_cnt_n) {
        LMB_CUDA(cudaStreamSynchronize(st));
        cudaFree(Z.prompt_cnt);
        Z.prompt_cnt = nullptr; Z.prompt_cnt_n = 0;
        LMB_TRY(dmalloc((void**)&Z.prompt_cnt, (int64_t)plan.n_counters * 4, true, st));
        Z.prompt_cnt_n = plan.n_counters;
      }
      LMB_TRY(window_attend(ctx, dt, b, q, plan, Z.prompt_part, Z.prompt_cnt, out, ldc, 0, st));
    }
    return LMB200_OK;
  };
  if (dt != LMB200_BF16 || graph || !flash_tc_window_supported(s.c.dim, s.c.vdim)) return split(0, T);
  auto flash = [&](int b, int n_batch, int t0, int n, int ctx_rows) -> int32_t {
    FlashWindowView f;
    f.H = v.H; f.G = v.H / v.G; f.dn = v.dim; f.dv = v.vdim; f.window = v.window; f.cap = v.score_cap;
    f.max_dot = 1.01f * v.dim;                                 // unit root mean squares, rounded to bf16
    f.q_s = qw; f.q_h = v.dim; f.q_b = (int64_t)n * qw;
    f.o_s = ldc; f.o_h = v.vdim; f.o_b = (int64_t)n * ldc;
    f.k_s = v.k_ld; f.k_h = (int64_t)v.cap * v.k_ld; f.k_b = v.G * f.k_h;
    f.v_s = v.v_ld; f.v_h = (int64_t)v.cap * v.v_ld; f.v_b = v.G * f.v_h;
    return flash_tc_launch_window(ctx, (char*)r.cat + (int64_t)t0 * ldc * e, (const char*)r.q + (int64_t)t0 * qw * e,
                                  (const char*)v.keys + b * f.k_b * e, (const char*)v.values + b * f.v_b * e, f, n_batch, n, ctx_rows, v.scale, st);
  };
  bool uniform = true;
  for (int b = 0; b < S->B; ++b) uniform = uniform && run.h_pos0[b] == run.h_pos0[0] && run.h_len[b] == run.h_len[0];
  if (uniform && run.h_len[0] >= kFlashMin && (int64_t)S->B * v.H <= 65535) return flash(0, S->B, 0, run.h_len[0], run.h_pos0[0] + run.h_len[0]);
  int pending = 0;
  for (int b = 0; b < S->B; ++b) {
    const int t0 = run.h_start[b], n = run.h_len[b];
    if (n < kFlashMin) continue;
    LMB_TRY(split(pending, t0));
    pending = t0 + n;
    LMB_TRY(flash(b, 1, t0, n, run.h_pos0[b] + n));
  }
  return split(pending, T);
}

int32_t delta_rows(Session* S, RowsBuf& r, const RowsRun& run, int l, cudaStream_t st) {
  Model* M = S->m;
  Ctx* ctx = M->ctx;
  const LayerSpec& s = M->specs[l];
  LayeredWeights& w = M->lw[l];
  const int dt = M->cfg.dtype, T = run.T, e = M->esz, ld_lr = row_ld(s.m_lr.K), ld_g = row_ld(out_width(s)), kd = s.c.kv_heads * s.c.dim, hd = s.c.heads * s.c.dim;
  char* proj = reinterpret_cast<char*>(r.proj);
  auto at = [&](int slot) { return (void*)(proj + (int64_t)s.row0[slot] * e); };
  RowSegs in;
  in.add(s.row0[D_Q], kd, SEG_ACT, at(D_Q), s.n_store);
  in.add(s.row0[D_K], kd, SEG_ACT, at(D_K), s.n_store);
  in.add(s.row0[D_V], out_width(s), SEG_ACT, at(D_V), s.n_store);
  in.add(s.row0[D_B], s.c.heads, SEG_F32, r.beta, s.c.heads);
  in.add(s.row0[D_A1], s.c.decay_rank, SEG_ACT, r.lr_in, ld_lr);
  in.add(s.row0[D_G1], s.c.gate_rank, SEG_ACT, (char*)r.lr_in + (int64_t)s.lr_g1 * e, ld_lr);
  LMB_TRY(rows_gemm(M, w.w_in, s.m_in, r.xn, row_ld(M->cfg.hidden), T, in, st));
  RowSegs lr;
  lr.add(s.m_lr.row_off[0], hd, SEG_DECAY, r.log_g, hd);
  lr.s[0].rate = w.a_log; lr.s[0].bias = w.dt_bias; lr.s[0].head = s.c.dim;
  lr.add(s.m_lr.row_off[1], out_width(s), SEG_SIGMOID, r.gate, ld_g);
  LMB_TRY(rows_gemm(M, w.w_lr, s.m_lr, r.lr_in, ld_lr, T, lr, st));
  DeltaView v = delta_view(S, l);
  v.start = run.start; v.len = run.len; v.pos0 = run.pos0; v.total = T; v.seq = run.seq; v.pos = run.pos;
  v.q = at(D_Q); v.k = at(D_K); v.v = at(D_V);
  v.q_pitch = v.k_pitch = v.v_pitch = s.n_store;
  LMB_TRY(delta_conv(ctx, dt, v, r.q, r.rq, r.rk, st));
  v.q = r.q; v.k = (char*)r.q + (int64_t)kd * e; v.v = (char*)r.q + (int64_t)2 * kd * e;
  v.q_pitch = v.k_pitch = v.v_pitch = delta_channels(s);
  v.rq = r.rq; v.rk = r.rk;
  v.b = r.beta; v.b_pitch = s.c.heads;
  v.decay = r.log_g; v.decay_pitch = hd;
  v.gate = r.gate; v.gate_pitch = ld_g;
  v.out = r.cat; v.ldo = row_ld(s.m_out.K); v.bp = 0;
  if (dt == LMB200_BF16 && run.max_len >= kDeltaTcMin && delta_tc_ok(v)) return delta_tc(ctx, v, st);
  if (dt == LMB200_BF16 && run.max_len >= kChunkMin && delta_chunks_ok(v)) return delta_chunks(ctx, v, st);
  return delta_steps(ctx, dt, v, st);
}

int32_t retention_rows(Session* S, RowsBuf& r, const RowsRun& run, int l, cudaStream_t st) {
  Model* M = S->m;
  Ctx* ctx = M->ctx;
  const LayerSpec& s = M->specs[l];
  LayeredWeights& w = M->lw[l];
  const int dt = M->cfg.dtype, T = run.T, e = M->esz, ldc = row_ld(s.m_out.K);
  // bf16: the projection's epilogue rotates q and k (pairs are neighbouring rows; heads of odd width are rotated by the consumer)
  const bool rot = dt == LMB200_BF16 && s.c.rot_dims > 0 && s.c.dim % 2 == 0, light = is_lightning(s);
  char* proj = reinterpret_cast<char*>(r.proj);
  auto at = [&](int slot) { return (void*)(proj + (int64_t)s.row0[slot] * e); };
  RowSegs in;
  const int kind = light ? SEG_SILU : rot ? SEG_ROT : SEG_ACT;
  in.add(s.row0[R_Q], s.c.heads * s.c.dim, kind, at(R_Q), s.n_store);
  in.add(s.row0[R_K], s.c.heads * s.c.dim, kind, at(R_K), s.n_store);
  if (rot)
    for (int i = 0; i < 2; ++i) LMB_TRY(rotate_segment(S, r, run, l, in.s[i], s.c.dim, 0, st));
  in.add(s.row0[R_V], out_width(s), light ? SEG_SILU : SEG_ACT, at(R_V), s.n_store);
  in.add(s.row0[R_G], out_width(s), light ? SEG_SIGMOID : SEG_SILU, at(R_G), s.n_store);
  if (s.c.ff && !post_norm(M)) in.add(s.row0[R_UP], s.c.ff, SEG_RELU2, (char*)r.cat + (int64_t)s.cat0 * e, ldc);
  LMB_TRY(rows_gemm(M, w.w_in, s.m_in, r.xn, row_ld(M->cfg.hidden), T, in, st));
  RetentionView v = retention_view(S, l);
  v.start = run.start; v.len = run.len; v.pos0 = run.pos0; v.total = run.T;
  v.q = at(R_Q); v.k = at(R_K); v.v = at(R_V); v.g = at(R_G);
  v.q_pitch = v.k_pitch = v.v_pitch = v.g_pitch = s.n_store;
  v.in_f32 = dt != LMB200_BF16; v.raw_gate = 0;
  v.out = r.cat; v.ldo = ldc; v.bp = 0;
  if (light) { v.ssq = r.ssq; v.ssq_t = s.c.heads; v.ssq_h = 1; }
  if (rot) v.rot_dims = 0;
  if (run.max_len >= kTcMin && retention_tc_ok(v)) return retention_tc(ctx, v, st);
  if (run.max_len >= kChunkMin && retention_chunks_ok(v)) return retention_chunks(ctx, v, st);
  return retention_steps(ctx, dt, v, st);
}

template <typename WT>
int32_t post_rows(Session* S, RowsBuf& r, const RowsRun& run, bool embed, const float* w, const LayerSpec* lightning, float* capture, cudaStream_t st) {
  const Model* M = S->m;
  const int W = M->cfg.hidden;
  LMB_CUDA(launch_k(rows_post_kernel<WT>, dim3((unsigned)run.T), dim3(256), (size_t)W * 4, st, r.x, (const float*)r.delta,
                    embed ? run.tokens : (const int*)nullptr, (const WT*)M->embed, M->cfg.vocab, M->embed_scale, w,
                    lightning ? (const float*)r.ssq : (const float*)nullptr, lightning ? lightning->c.heads : 0, lightning ? out_width(*lightning) : 1, (WT*)r.xn,
                    row_ld(W), W, M->cfg.rms_eps, capture, run.last));
  M->ctx->launches++;
  return LMB200_OK;
}

// the sublayers of layer l one after another, each normed on its output; x and xn (its copy in the model dtype) hold the residual rows
template <typename WT>
int32_t post_layer(Session* S, RowsBuf& r, const RowsRun& run, int l, bool graph, cudaStream_t st) {
  Model* M = S->m;
  Ctx* ctx = M->ctx;
  const LayerSpec& s = M->specs[l];
  LayeredWeights& w = M->lw[l];
  const int W = M->cfg.hidden, T = run.T, ldx = row_ld(W), e = M->esz, last = M->side_dim ? 2 : s.c.ff ? 1 : 0;
  float* cap = S->capture_on ? S->capture + (int64_t)l * S->B * W : nullptr;
  RowSegs out;
  out.add(0, W, SEG_F32, r.delta, W);
  LMB_TRY(is_attention(s) ? attention_rows(S, r, run, l, graph, st) : is_delta(s) ? delta_rows(S, r, run, l, st) : retention_rows(S, r, run, l, st));
  LMB_TRY(rows_gemm(M, w.w_out, s.m_out, r.cat, row_ld(s.m_out.K), T, out, st));
  LMB_TRY(post_rows<WT>(S, r, run, false, w.norm, is_lightning(s) ? &s : nullptr, last == 0 ? cap : nullptr, st));
  if (s.c.ff) {
    const int lda = row_ld(s.c.ff);
    if (e == 2) {
      LMB_TRY(gemm_silu_gate_bf16(ctx, w.w_gu, r.xn, ldx, T, s.m_gu.rows, s.m_gu.K, r.act, lda, s.c.ff, st));
    } else {
      RowSegs gu;
      gu.add(0, s.m_gu.rows, SEG_F32, r.proj, s.m_gu.rows);
      LMB_TRY(rows_gemm(M, w.w_gu, s.m_gu, r.xn, ldx, T, gu, st));
      LMB_CUDA(launch_k(silu_gate_rows_kernel, dim3((unsigned)std::min<int64_t>(ceil_div((int64_t)T * s.c.ff, 256), 16 * ctx->sm_count)), dim3(256), 0, st,
                        (const float*)r.proj, s.m_gu.rows, (float*)r.act, lda, s.c.ff, T));
      ctx->launches++;
    }
    LMB_TRY(rows_gemm(M, w.w_down, s.m_down, r.act, lda, T, out, st));
    LMB_TRY(post_rows<WT>(S, r, run, false, w.norm2, nullptr, last == 1 ? cap : nullptr, st));
  }
  if (M->side_dim) {
    const int lds = row_ld(M->side_dim);
    RowSegs g;
    g.add(0, M->side_dim, SEG_GELU_TOKEN, r.side, lds);
    g.s[0].table = (const char*)M->side_embed + (int64_t)l * M->side_dim * e;
    g.s[0].table_pitch = M->cfg.n_layers * M->side_dim; g.s[0].table_rows = M->cfg.vocab; g.s[0].tokens = run.tokens;
    LMB_TRY(rows_gemm(M, w.w_sg, s.m_sg, r.xn, ldx, T, g, st));
    LMB_TRY(rows_gemm(M, w.w_sp, s.m_sp, r.side, lds, T, out, st));
    LMB_TRY(post_rows<WT>(S, r, run, false, w.side_norm, nullptr, cap, st));
  }
  return LMB200_OK;
}

// one pass over packed tokens; the residual rows of the last layer are left in x + delta (in x where outputs are captured or the
// sublayers are normed on their output)
int32_t rows_step(Session* S, RowsBuf& r, const RowsRun& run, bool graph, cudaStream_t st) {
  Model* M = S->m;
  const int W = M->cfg.hidden, L = M->cfg.n_layers, bf = M->cfg.dtype == LMB200_BF16;
  r.packed_layer = -1;
  r.angles_valid.assign(M->rot_freqs.size(), false);
  if (post_norm(M)) {
    LMB_TRY(bf ? post_rows<__nv_bfloat16>(S, r, run, true, nullptr, nullptr, nullptr, st) : post_rows<float>(S, r, run, true, nullptr, nullptr, nullptr, st));
    for (int l = 0; l < L; ++l) LMB_TRY(bf ? post_layer<__nv_bfloat16>(S, r, run, l, graph, st) : post_layer<float>(S, r, run, l, graph, st));
    return LMB200_OK;
  }
  for (int l = 0; l < L; ++l) {
    float* cap = S->capture_on && l > 0 ? S->capture + (int64_t)(l - 1) * S->B * W : nullptr;
    const float* delta = l ? r.delta : nullptr;
    LMB_TRY(bf ? norm_rows<__nv_bfloat16>(S, r, run, run.T, delta, l == 0, nullptr, M->lw[l].norm, r.xn, cap, st)
               : norm_rows<float>(S, r, run, run.T, delta, l == 0, nullptr, M->lw[l].norm, r.xn, cap, st));
    const LayerSpec& s = M->specs[l];
    LMB_TRY(is_latent(s) ? latent_rows(S, r, run, l, graph, st) : retention_rows(S, r, run, l, st));
    RowSegs out;
    out.add(0, W, SEG_F32, r.delta, W);
    LMB_TRY(rows_gemm(M, M->lw[l].w_out, s.m_out, r.cat, row_ld(s.m_out.K), run.T, out, st));
  }
  if (S->capture_on) {
    float* cap = S->capture + (int64_t)(L - 1) * S->B * W;
    LMB_TRY(norm_rows<float>(S, r, run, run.T, r.delta, false, nullptr, nullptr, nullptr, cap, st));
  }
  return LMB200_OK;
}

// final norm and head on the rows `pick` chooses: logits [n, pitch]
int32_t rows_head(Session* S, RowsBuf& r, const RowsRun& run, const int* pick, int n, void* xn, float* logits, int pitch, cudaStream_t st) {
  Model* M = S->m;
  const int W = M->cfg.hidden;
  const float* delta = S->capture_on || post_norm(M) ? nullptr : r.delta;
  LMB_TRY(M->cfg.dtype == LMB200_BF16 ? norm_rows<__nv_bfloat16>(S, r, run, n, delta, false, pick, M->final_norm, xn, nullptr, st)
                                      : norm_rows<float>(S, r, run, n, delta, false, pick, M->final_norm, xn, nullptr, st));
  RowSegs h;
  h.add(0, M->cfg.vocab, SEG_SOFTCAP, logits, pitch);
  h.softcap = M->softcap;
  return rows_gemm(M, M->lm_head, M->m_head, xn, row_ld(W), n, h, st);
}

// bf16, one token per sequence, sublayers normed on their output
int32_t fused_post_step(Session* S, cudaStream_t st, bool with_head) {
  Model* M = S->m;
  Ctx* ctx = M->ctx;
  LayeredScratch& Z = *S->lay;
  const int B = S->B, hid = M->cfg.hidden, L = M->cfg.n_layers, dt = LMB200_BF16;
  int tiles = 1;                                             // CTAs of the last output projection
  // Slots of the step's n_post output norms: two sets in turn, and a third for the last of an odd number, so that a launch and the
  // one after it (the step is replayed) never share a set
  int n_post = 0, at_post = 0;
  for (const LayerSpec& s : M->specs) n_post += 1 + (s.c.ff > 0) + (M->side_dim > 0);
  auto slots = [&](int i) { return Z.post_slots + (int64_t)(n_post % 2 && i == n_post - 1 ? 2 : i & 1) * kPushMaxCtas * 32; };
  // the matrix that follows: its weights are drawn into L2 while this one drains
  struct Next { const void* W = nullptr; const WMap* m = nullptr; const GemvPlan* pl = nullptr; };
  auto launch = [&](GemvParams& p, const Next& nx) -> int32_t {
    if (nx.W) gemv_prefetch_next(p, ctx, dt, nx.W, nx.m->rows, nx.m->K, *nx.pl);
    return gemv_launch(ctx, dt, p, st);
  };
  auto head_next = [&]() { Next n; if (with_head) { n.W = M->lm_head; n.m = &M->m_head; n.pl = &S->p_head; } return n; };
  auto after = [&](int l) { Next n; if (l + 1 == L) return head_next(); n.W = M->lw[l + 1].w_in; n.m = &M->specs[l + 1].m_in; n.pl = &Z.p_in[l + 1]; return n; };
  // an output projection: residual += its norm; the last one of the step also prepares the final norm
  auto post = [&](int l, const void* W, const WMap& m, const GemvPlan& pl, const void* x, const float* w, InvScale iv, bool layer_end, const Next& nx) -> int32_t {
    GemvParams p = gemv_params(S, W, m, pl, x);
    p.epi = EPI_POST_NORM; p.inv = iv;
    p.pn.x = S->xT; p.pn.w = w; p.pn.xg = S->xn; p.pn.eps = M->cfg.rms_eps;
    p.pn.slots = slots(at_post); p.pn.clear = n_post > 1 ? slots((at_post + 1) % n_post) : nullptr;
    if (n_post == 1) LMB_CUDA(cudaMemsetAsync(p.pn.slots, 0xFF, (size_t)kPushMaxCtas * 32 * 4, st));
    ++at_post;
    if (layer_end && S->capture_on) p.pn.capture = S->capture + (int64_t)l * B * hid;
    if (layer_end && l + 1 == L) { p.pn.gain = M->final_norm; p.pn.ssq = S->ssq; }
    tiles = gemv_plan_ctas(pl, m.rows);
    return launch(p, nx);
  };
  LMB_TRY(embed_prep_launch(S, nullptr, st, M->embed_scale));
  for (int l = 0; l < L; ++l) {
    const LayerSpec& s = M->specs[l];
    LayeredWeights& w = M->lw[l];
    const bool ff = s.c.ff > 0, side = M->side_dim > 0, delta = is_delta(s);
    const Next out{w.w_out, &s.m_out, &Z.p_out[l]}, lr{w.w_lr, &s.m_lr, &Z.p_lr[l]}, gu{w.w_gu, &s.m_gu, &Z.p_gu[l]}, down{w.w_down, &s.m_down, &Z.p_down[l]};
    const Next sg{w.w_sg, &s.m_sg, &Z.p_sg[l]}, sp{w.w_sp, &s.m_sp, &Z.p_sp[l]};
    {
      GemvParams p = gemv_params(S, w.w_in, s.m_in, Z.p_in[l], S->xn);
      p.epi = EPI_STORE_F32; p.out = Z.proj; p.out_pitch = s.n_store;
      if (delta) { p.epi = EPI_STORE_ACT; p.act_row0 = s.n_store; p.act = Z.lr_in; p.act_col0 = 0; p.n_act = s.m_lr.K; }
      LMB_TRY(launch(p, delta ? lr : out));
    }
    InvScale iv;
    if (is_attention(s)) {
      WindowView v = window_view(S, l);
      v.T = B; v.seq = Z.iota; v.pos = S->pos;
      WindowRows in;
      in.q = Z.proj + s.row0[D_Q]; in.q_pitch = s.n_store; in.in_f32 = 1;
      if (s.c.kv_from < 0) {
        in.k = Z.proj + s.row0[D_K]; in.v = Z.proj + s.row0[D_V];
        in.k_pitch = in.v_pitch = s.n_store;
      }
      if (Z.win[l].nsplit == 0) {
        LMB_TRY(window_prep(ctx, dt, v, in, Z.qw, st));
        in.q = Z.qw; in.q_pitch = s.c.heads * s.c.dim; in.in_f32 = 0;
      }
      LMB_TRY(window_attend(ctx, dt, v, in, Z.win[l], Z.attn_part, Z.win_cnt, S->act, 0, S->Bp, st));
    } else if (delta) {
      GemvParams p = gemv_params(S, w.w_lr, s.m_lr, Z.p_lr[l], Z.lr_in);
      p.epi = EPI_STORE_F32; p.out = Z.lr; p.out_pitch = s.m_lr.rows;
      LMB_TRY(launch(p, out));
      DeltaView v = delta_view(S, l);
      v.start = Z.iota; v.len = Z.ones; v.pos0 = S->pos; v.total = B; v.raw = 1;
      v.q = Z.proj + s.row0[D_Q]; v.k = Z.proj + s.row0[D_K]; v.v = Z.proj + s.row0[D_V];
      v.q_pitch = v.k_pitch = v.v_pitch = v.b_pitch = s.n_store;
      v.b = Z.proj + s.row0[D_B];
      v.decay = Z.lr + s.m_lr.row_off[0]; v.gate = Z.lr + s.m_lr.row_off[1];
      v.decay_pitch = v.gate_pitch = s.m_lr.rows;
      v.out = S->act; v.bp = S->Bp;
      LMB_TRY(delta_steps(ctx, dt, v, st));
    } else {
      RetentionView v = retention_view(S, l);
      v.start = Z.iota; v.len = Z.ones; v.pos0 = S->pos;
      v.q = Z.proj + s.row0[R_Q]; v.k = Z.proj + s.row0[R_K]; v.v = Z.proj + s.row0[R_V]; v.g = Z.proj + s.row0[R_G];
      v.q_pitch = v.k_pitch = v.v_pitch = v.g_pitch = s.n_store;
      v.in_f32 = 1; v.raw_act = 1; v.raw_gate = 2;
      v.ssq = Z.mix_ssq; v.ssq_t = 1; v.ssq_h = 32;
      v.out = S->act; v.bp = S->Bp;
      LMB_TRY(retention_steps(ctx, dt, v, st));
      iv.ssq = Z.mix_ssq; iv.tiles = s.c.heads; iv.n = out_width(s); iv.eps = M->cfg.rms_eps;
    }
    LMB_TRY(post(l, w.w_out, s.m_out, Z.p_out[l], S->act, w.norm, iv, !ff && !side, ff ? gu : side ? sg : after(l)));
    if (ff) {
      GemvParams p = gemv_params(S, w.w_gu, s.m_gu, Z.p_gu[l], S->xn);
      p.epi = EPI_SILU_GATE; p.act = Z.act_ff; p.n_act = s.c.ff;
      LMB_TRY(launch(p, down));
      LMB_TRY(post(l, w.w_down, s.m_down, Z.p_down[l], Z.act_ff, w.norm2, InvScale(), !side, side ? sg : after(l)));
    }
    if (side) {
      GemvParams p = gemv_params(S, w.w_sg, s.m_sg, Z.p_sg[l], S->xn);
      p.epi = EPI_GELU_TOKEN; p.act = Z.act_side;
      p.token_table = (const __nv_bfloat16*)M->side_embed + (int64_t)l * M->side_dim; p.token_pitch = L * M->side_dim; p.token_rows = M->cfg.vocab; p.tokens = S->tokens;
      LMB_TRY(launch(p, sp));
      LMB_TRY(post(l, w.w_sp, s.m_sp, Z.p_sp[l], Z.act_side, w.side_norm, InvScale(), true, after(l)));
    }
  }
  if (with_head) {
    GemvParams p = gemv_params(S, M->lm_head, M->m_head, S->p_head, S->xn);
    p.epi = EPI_STORE_F32; p.out = S->logits; p.out_pitch = S->logits_pitch; p.softcap = M->softcap;
    p.inv.ssq = S->ssq; p.inv.tiles = tiles; p.inv.n = hid; p.inv.eps = M->cfg.rms_eps;
    LMB_TRY(gemv_launch(ctx, dt, p, st));
  }
  return LMB200_OK;
}

// bf16, one token per sequence
int32_t fused_step(Session* S, cudaStream_t st, bool with_head) {
  Model* M = S->m;
  Ctx* ctx = M->ctx;
  LayeredScratch& Z = *S->lay;
  const int B = S->B, hid = M->cfg.hidden, L = M->cfg.n_layers, dt = LMB200_BF16;
  LMB_TRY(embed_prep_launch(S, M->lw[0].norm, st));
  int tiles = (int)ceil_div(hid, S->embed_rows_per_cta);
  auto inv_scale = [&]() { InvScale iv; iv.ssq = S->ssq; iv.tiles = tiles; iv.n = hid; iv.eps = M->cfg.rms_eps; return iv; };
  for (int l = 0; l < L; ++l) {
    const LayerSpec& s = M->specs[l];
    LayeredWeights& w = M->lw[l];
    {
      GemvParams p = gemv_params(S, w.w_in, s.m_in, Z.p_in[l], S->xn);
      p.epi = EPI_STORE_RELU2; p.inv = inv_scale();
      p.out = Z.proj; p.out_pitch = s.n_store; p.act_row0 = s.n_store; p.act = S->act; p.act_col0 = s.cat0; p.n_act = s.c.ff;
      if (is_latent(s)) gemv_prefetch_next(p, ctx, dt, w.w_uq, s.m_uq.rows, s.m_uq.K, Z.p_uq[l]);
      else gemv_prefetch_next(p, ctx, dt, w.w_out, s.m_out.rows, s.m_out.K, Z.p_out[l]);
      LMB_TRY(gemv_launch(ctx, dt, p, st));
    }
    if (is_latent(s)) {
      const bool own = s.c.kv_from < 0;
      LatentView v = latent_view(S, l);
      v.T = B; v.seq = Z.iota; v.pos = S->pos;
      void* cache = S->latent[cache_layer(M, l)];
      LMB_TRY(latent_prep(ctx, dt, v, Z.proj, s.n_store, s.row0[L_DQ], own ? s.row0[L_DKV] : 0, w.q_norm, w.kv_norm, Z.xq, 0, S->Bp,
                          own ? cache : nullptr, nullptr, st));
      GemvParams p = gemv_params(S, w.w_uq, s.m_uq, Z.p_uq[l], Z.xq);
      p.epi = EPI_STORE_F32; p.out = Z.qf; p.out_pitch = q_width(s);
      gemv_prefetch_next(p, ctx, dt, w.w_out, s.m_out.rows, s.m_out.K, Z.p_out[l]);
      LMB_TRY(gemv_launch(ctx, dt, p, st));
      LMB_TRY(latent_absorb(ctx, dt, v, Z.qf, 1, w.w_ukt, Z.qa, st));
      LMB_TRY(latent_attend(ctx, dt, v, Z.qa, cache, Z.attn[l], Z.attn_part, st));
      LMB_TRY(latent_expand(ctx, dt, v, Z.attn_part, Z.attn[l], w.w_uv, Z.proj + s.row0[L_G], s.n_store, S->act, 0, S->Bp, st));
    } else {
      RetentionView v = retention_view(S, l);
      v.start = Z.iota; v.len = Z.ones; v.pos0 = S->pos;
      v.q = Z.proj + s.row0[R_Q]; v.k = Z.proj + s.row0[R_K]; v.v = Z.proj + s.row0[R_V]; v.g = Z.proj + s.row0[R_G];
      v.q_pitch = v.k_pitch = v.v_pitch = v.g_pitch = s.n_store;
      v.in_f32 = 1; v.raw_gate = 1;
      v.out = S->act; v.bp = S->Bp;
      LMB_TRY(retention_steps(ctx, dt, v, st));
    }
    {
      GemvParams p = gemv_params(S, w.w_out, s.m_out, Z.p_out[l], S->act);
      p.epi = EPI_RESID_NORM;
      p.rn.x = S->xT; p.rn.gain = l + 1 < L ? M->lw[l + 1].norm : M->final_norm; p.rn.xg = S->xn; p.rn.ssq = S->ssq;
      p.rn.capture = S->capture_on ? S->capture + (int64_t)l * B * hid : nullptr;
      if (l + 1 < L) gemv_prefetch_next(p, ctx, dt, M->lw[l + 1].w_in, M->specs[l + 1].m_in.rows, M->specs[l + 1].m_in.K, Z.p_in[l + 1]);
      else if (with_head) gemv_prefetch_next(p, ctx, dt, M->lm_head, M->m_head.rows, M->m_head.K, S->p_head);
      LMB_TRY(gemv_launch(ctx, dt, p, st));
      tiles = gemv_plan_ctas(Z.p_out[l], s.m_out.rows);
    }
  }
  if (with_head) {
    GemvParams p = gemv_params(S, M->lm_head, M->m_head, S->p_head, S->xn);
    p.epi = EPI_STORE_F32; p.inv = inv_scale(); p.out = S->logits; p.out_pitch = S->logits_pitch; p.softcap = M->softcap;
    LMB_TRY(gemv_launch(ctx, dt, p, st));
  }
  return LMB200_OK;
}

RowsRun decode_run(const Session* S) {
  const LayeredScratch& Z = *S->lay;
  RowsRun run;
  run.T = S->B;
  run.tokens = S->tokens; run.seq = Z.iota; run.pos = S->pos; run.last = Z.iota;
  run.start = Z.iota; run.len = Z.ones; run.pos0 = S->pos;
  run.ctx_len = S->cap;
  return run;
}

int32_t ensure_want(Session* S, int64_t n) {
  LayeredScratch& Z = *S->lay;
  if (n <= Z.want_cap) return LMB200_OK;
  cudaFree(Z.want_logits); cudaFree(Z.want_xn);
  Z.want_logits = nullptr; Z.want_xn = nullptr; Z.want_cap = 0;
  LMB_TRY(dmalloc((void**)&Z.want_logits, n * S->m->cfg.vocab * 4, false, S->m->ctx->stream));
  LMB_TRY(dmalloc(&Z.want_xn, n * row_ld(S->m->cfg.hidden) * S->m->esz, true, S->m->ctx->stream));
  Z.want_cap = n;
  return LMB200_OK;
}

}  // namespace

int32_t layered_enqueue_step(Session* S, cudaStream_t st, bool with_head) {
  if (S->m->cfg.dtype == LMB200_BF16) {
    LMB_TRY(post_norm(S->m) ? fused_post_step(S, st, with_head) : fused_step(S, st, with_head));
  } else {
    LayeredScratch& Z = *S->lay;
    const RowsRun run = decode_run(S);
    LMB_TRY(rows_step(S, Z.step, run, true, st));
    if (with_head) LMB_TRY(rows_head(S, Z.step, run, Z.iota, S->B, Z.step.xn, S->logits, S->logits_pitch, st));
  }
  if (with_head) LMB_TRY(argmax_launch(S, st));
  return advance_launch(S, st);
}

int32_t layered_session_create(Model* M, int batch, int max_ctx, lmb200_session* out) {
  Ctx* ctx = M->ctx;
  LMB_CUDA(cudaSetDevice(ctx->device));
  const lmb200_model_config& c = M->cfg;
  const bool bf = c.dtype == LMB200_BF16;
  Session* S = new Session();
  S->m = M; S->B = batch; S->max_ctx = max_ctx;
  S->cap = (int)round_up(max_ctx, 64);
  S->Bp = bf ? Layout<__nv_bfloat16>::batch_pad(batch) : Layout<float>::batch_pad(batch);
  S->logits_pitch = (int)round_up(c.vocab, 16);
  S->lay = new LayeredScratch();
  LayeredScratch& Z = *S->lay;
  int32_t rc = LMB200_OK;
  auto alloc = [&](void** p, int64_t bytes) { if (rc == LMB200_OK) rc = dmalloc(p, bytes, true, ctx->stream); };
  S->latent.assign(c.n_layers, nullptr);
  S->state.assign(c.n_layers, nullptr);
  S->keys.assign(c.n_layers, nullptr);
  S->values.assign(c.n_layers, nullptr);
  S->conv.assign(c.n_layers, nullptr);
  int64_t lat_parts = 0, win_units = 0;
  for (int l = 0; l < c.n_layers; ++l) {
    const LayerSpec& s = M->specs[l];
    if (is_attention(s)) {
      if (s.c.kv_from >= 0) continue;
      alloc(&S->keys[l], (int64_t)batch * s.c.kv_heads * S->cap * s.k_ld * M->esz);
      alloc(&S->values[l], (int64_t)batch * s.c.kv_heads * S->cap * s.v_ld * M->esz);
      continue;
    }
    if (is_delta(s)) alloc((void**)&S->conv[l], (int64_t)batch * s.c.conv * delta_channels(s) * 4);
    if (!is_latent(s)) { alloc((void**)&S->state[l], (int64_t)batch * s.c.heads * s.c.dim * state_ld(s) * 4); continue; }
    if (s.c.kv_from < 0) alloc(&S->latent[l], (int64_t)batch * S->cap * s.lat_ld * M->esz);
  }
  Z.attn.resize(c.n_layers);
  Z.win.resize(c.n_layers);
  for (int l = 0; l < c.n_layers; ++l) {
    const LayerSpec& s = M->specs[l];
    if (is_attention(s)) {
      Z.win[l] = window_plan(ctx, c.dtype, window_view(S, l), batch, S->cap);
      lat_parts = std::max(lat_parts, Z.win[l].part_floats);
      win_units = std::max<int64_t>(win_units, Z.win[l].n_counters);
    }
    if (!is_latent(s)) continue;
    Z.attn[l] = latent_attn_plan(ctx, c.dtype, latent_view(S, l), batch, S->cap);
    lat_parts = std::max(lat_parts, Z.attn[l].part_floats);
  }
  if (bf) {
    int64_t max_part = 0;
    int max_cnt = 0;
    auto take = [&](const GemvPlan& g) { max_part = std::max(max_part, g.partial_floats); max_cnt = std::max(max_cnt, g.n_counters); return g; };
    for (const LayerSpec& s : M->specs) {
      Z.p_in.push_back(take(gemv_plan(ctx, c.dtype, batch, s.m_in.rows, s.m_in.K)));
      Z.p_uq.push_back(is_latent(s) ? take(gemv_plan(ctx, c.dtype, batch, s.m_uq.rows, s.m_uq.K)) : GemvPlan());
      Z.p_out.push_back(take(gemv_plan_resid(ctx, batch, s.m_out.rows, s.m_out.K)));
      if (Z.p_out.back().cluster < 1 && rc == LMB200_OK) rc = fail(LMB200_EINVAL, "session_create: width %d has more than one wave of row groups", c.hidden);
      const bool ff = post_norm(M) && s.c.ff > 0, side = M->side_dim > 0;
      Z.p_gu.push_back(ff ? take(gemv_plan(ctx, c.dtype, batch, s.m_gu.rows, s.m_gu.K)) : GemvPlan());
      Z.p_down.push_back(ff ? take(gemv_plan_resid(ctx, batch, s.m_down.rows, s.m_down.K)) : GemvPlan());
      Z.p_sg.push_back(side ? take(gemv_plan(ctx, c.dtype, batch, s.m_sg.rows, s.m_sg.K)) : GemvPlan());
      Z.p_sp.push_back(side ? take(gemv_plan_resid(ctx, batch, s.m_sp.rows, s.m_sp.K)) : GemvPlan());
      Z.p_lr.push_back(is_delta(s) ? take(gemv_plan(ctx, c.dtype, batch, s.m_lr.rows, s.m_lr.K)) : GemvPlan());
    }
    S->p_head = take(gemv_plan(ctx, c.dtype, batch, M->m_head.rows, M->m_head.K));
    S->embed_rows_per_cta = 32 * (int)ceil_div(c.hidden, 32 * 256);
    auto x_bytes = [&](int64_t K) { return Layout<__nv_bfloat16>::x_elems((int)K, S->Bp) * 2; };
    alloc(&S->xn, x_bytes(c.hidden));
    alloc(&S->act, x_bytes(max_over(M, [](const LayerSpec& s) { return s.m_out.K; })));
    alloc((void**)&S->xT, (int64_t)round_up(c.hidden, 128) * S->Bp * 4);
    alloc((void**)&S->ssq, (int64_t)256 * 32 * 4);
    alloc((void**)&S->gemv_partials, max_part * 4);
    alloc((void**)&S->gemv_counters, (int64_t)max_cnt * 4);
    alloc((void**)&Z.proj, batch * max_over(M, [](const LayerSpec& s) { return s.n_store; }) * 4);
    alloc((void**)&Z.qf, batch * max_over(M, [](const LayerSpec& s) { return is_latent(s) ? q_width(s) : 0; }) * 4);
    alloc(&Z.xq, x_bytes(std::max<int64_t>(1, max_over(M, [](const LayerSpec& s) { return s.c.q_rank; }))));
    alloc(&Z.qa, batch * max_over(M, [](const LayerSpec& s) { return is_latent(s) ? (int64_t)s.c.heads * s.lat_ld : 0; }) * 2);
    if (post_norm(M)) {
      const int64_t qw = max_over(M, [&](const LayerSpec& s) { return is_attention(s) ? (int64_t)s.c.heads * s.c.dim : 0; });
      alloc(&Z.act_ff, x_bytes(std::max<int64_t>(1, max_over(M, [](const LayerSpec& s) { return s.c.ff; }))));
      alloc(&Z.act_side, x_bytes(std::max(1, M->side_dim)));
      alloc(&Z.lr_in, x_bytes(std::max<int64_t>(1, max_over(M, [](const LayerSpec& s) { return s.m_lr.K; }))));
      alloc((void**)&Z.lr, batch * max_over(M, [](const LayerSpec& s) { return s.m_lr.rows; }) * 4);
      alloc((void**)&Z.mix_ssq, max_over(M, [](const LayerSpec& s) { return is_lightning(s) ? s.c.heads : 0; }) * 32 * 4);
      alloc((void**)&Z.post_slots, (int64_t)3 * kPushMaxCtas * 32 * 4);
      if (rc == LMB200_OK && cudaMemsetAsync(Z.post_slots, 0xFF, (size_t)3 * kPushMaxCtas * 32 * 4, ctx->stream) != cudaSuccess)
        rc = fail(LMB200_ECUDA, "session_create: memset failed");
      alloc(&Z.qw, batch * qw * 2);
    }
    S->fused = true;
  } else if (rc == LMB200_OK) {
    rc = ensure_rows(S, Z.step, batch, 0);
  }
  alloc((void**)&Z.attn_part, lat_parts * 4);
  alloc((void**)&Z.win_cnt, win_units * 4);
  alloc((void**)&S->logits, (int64_t)batch * S->logits_pitch * 4);
  alloc((void**)&S->tokens, (int64_t)batch * 4);
  alloc((void**)&S->pos, (int64_t)batch * 4);
  alloc((void**)&S->limit, (int64_t)batch * 4);
  alloc((void**)&S->step_ctr, 4);
  alloc((void**)&S->stop, (int64_t)(2 + batch) * 4);
  alloc((void**)&S->tok_hist, (int64_t)(S->cap + 1) * batch * 4);
  alloc((void**)&Z.iota, (int64_t)batch * 4);
  alloc((void**)&Z.ones, (int64_t)batch * 4);
  S->host_pos_v.assign(batch, 0);
  if (rc == LMB200_OK) {
    std::vector<int> iota(batch), ones(batch, 1), limit(batch, 0x7fffffff);
    for (int b = 0; b < batch; ++b) iota[b] = b;
    const int no_eot = -1;
    const bool ok = cudaMemcpyAsync(Z.iota, iota.data(), batch * 4, cudaMemcpyHostToDevice, ctx->stream) == cudaSuccess &&
                    cudaMemcpyAsync(Z.ones, ones.data(), batch * 4, cudaMemcpyHostToDevice, ctx->stream) == cudaSuccess &&
                    cudaMemcpyAsync(S->limit, limit.data(), batch * 4, cudaMemcpyHostToDevice, ctx->stream) == cudaSuccess &&
                    cudaMemcpyAsync(S->stop, &no_eot, 4, cudaMemcpyHostToDevice, ctx->stream) == cudaSuccess &&
                    cudaStreamSynchronize(ctx->stream) == cudaSuccess;
    if (!ok) rc = fail(LMB200_ECUDA, "session_create: upload failed");
  }
  if (rc != LMB200_OK) { lmb200_session_destroy(reinterpret_cast<lmb200_session>(S)); return rc; }
  *out = reinterpret_cast<lmb200_session>(S);
  return LMB200_OK;
}

void layered_session_free(Session* S) {
  for (void* p : S->latent) cudaFree(p);
  for (float* p : S->state) cudaFree(p);
  for (void* p : S->keys) cudaFree(p);
  for (void* p : S->values) cudaFree(p);
  for (float* p : S->conv) cudaFree(p);
  S->latent.clear();
  S->state.clear();
  S->keys.clear();
  S->values.clear();
  S->conv.clear();
  if (!S->lay) return;
  LayeredScratch& Z = *S->lay;
  cudaFree(Z.proj); cudaFree(Z.qf); cudaFree(Z.xq); cudaFree(Z.qa); cudaFree(Z.iota); cudaFree(Z.ones);
  cudaFree(Z.attn_part); cudaFree(Z.prompt_part); cudaFree(Z.win_cnt); cudaFree(Z.prompt_cnt);
  cudaFree(Z.act_ff); cudaFree(Z.act_side); cudaFree(Z.lr_in); cudaFree(Z.qw); cudaFree(Z.lr); cudaFree(Z.mix_ssq); cudaFree(Z.post_slots);
  cudaFree(Z.want_logits); cudaFree(Z.want_xn); cudaFree(Z.expanded);
  free_rows(Z.step);
  free_rows(Z.prompt);
  delete S->lay;
  S->lay = nullptr;
}

int32_t layered_check_positions(const Session* S, const int32_t* pos) {
  if (!layered_has_state(S->m)) return LMB200_OK;
  for (int b = 0; b < S->B; ++b)
    if (pos[b] != 0 && pos[b] != S->host_pos_v[b])
      return fail(LMB200_ESTATE, "set_position: sequence %d is at %d; its recurrent state cannot be moved to position %d (0 empties it)", b,
                  S->host_pos_v[b], pos[b]);
  return LMB200_OK;
}

int32_t layered_clear_state(Session* S, const int32_t* new_pos) {
  const Model* M = S->m;
  for (int l = 0; l < M->cfg.n_layers; ++l) {
    if (!S->state[l]) continue;
    const LayerSpec& s = M->specs[l];
    const int64_t per = (int64_t)s.c.heads * s.c.dim * state_ld(s);
    for (int b = 0; b < S->B; ++b)
      if (new_pos[b] == 0) LMB_CUDA(cudaMemsetAsync(S->state[l] + b * per, 0, (size_t)per * 4, M->ctx->stream));
  }
  return LMB200_OK;
}

int32_t layered_fill_random(Session* S, int32_t n_pos, uint64_t seed) {
  Model* M = S->m;
  const float scale = 1.0f / 131072.0f;
  for (int l = 0; l < M->cfg.n_layers; ++l) {
    const LayerSpec& s = M->specs[l];
    const uint64_t key = stream_key(seed, kIdLayeredState + l);
    if (S->keys[l]) {
      for (int i = 0; i < S->B * s.c.kv_heads && n_pos > 0; ++i) {
        LMB_TRY(fill_plain_dt(M, M->cfg.dtype, (char*)S->keys[l] + (int64_t)i * S->cap * s.k_ld * M->esz, n_pos, s.k_ld, key + 2 * i, nullptr, 0, scale, 0.f));
        LMB_TRY(fill_plain_dt(M, M->cfg.dtype, (char*)S->values[l] + (int64_t)i * S->cap * s.v_ld * M->esz, n_pos, s.v_ld, key + 2 * i + 1, nullptr, 0, scale, 0.f));
      }
    } else if (S->latent[l]) {
      if (n_pos == 0) continue;
      for (int b = 0; b < S->B; ++b) {
        char* base = reinterpret_cast<char*>(S->latent[l]) + (int64_t)b * S->cap * s.lat_ld * M->esz;
        LMB_TRY(fill_plain_dt(M, M->cfg.dtype, base, n_pos, s.lat_ld, key + b, nullptr, 0, scale, 0.f));
      }
    } else if (S->state[l]) {
      const int64_t rows = (int64_t)S->B * s.c.heads * s.c.dim;
      if (n_pos == 0) LMB_CUDA(cudaMemsetAsync(S->state[l], 0, (size_t)(rows * state_ld(s)) * 4, M->ctx->stream));
      else LMB_TRY(fill_plain_dt(M, LMB200_F32, S->state[l], rows, state_ld(s), key, nullptr, 0, scale, 0.f));
      if (S->conv[l]) LMB_TRY(fill_plain_dt(M, LMB200_F32, S->conv[l], (int64_t)S->B * s.c.conv, delta_channels(s), key + 1, nullptr, 0, scale, 0.f));
    }
  }
  return LMB200_OK;
}

int32_t layered_extend(Session* S, const int32_t* tokens, const int32_t* lengths, int32_t n_want, const int32_t* want, float* logits_out,
                       bool greedy) {
  Model* M = S->m;
  Ctx* ctx = M->ctx;
  LayeredScratch& Z = *S->lay;
  const int B = S->B, V = M->cfg.vocab;
  LMB_CUDA(cudaSetDevice(ctx->device));
  int T = 0, max_len = 0, ctx_len = 0;
  bool single = true;
  for (int b = 0; b < B; ++b) {
    T += lengths[b];
    max_len = std::max(max_len, lengths[b]);
    ctx_len = std::max(ctx_len, S->host_pos_v[b] + lengths[b]);
    single = single && lengths[b] == 1;
  }
  LMB_CUDA(cudaMemsetAsync(S->step_ctr, 0, 4, ctx->stream));
  if (single) {                                   // the decode step
    LMB_CUDA(cudaMemcpyAsync(S->tokens, tokens, (size_t)B * 4, cudaMemcpyHostToDevice, ctx->stream));
    LMB_TRY(run_step(S, n_want > 0, logits_out != nullptr));
    for (int i = 0; i < n_want && logits_out; ++i)
      LMB_CUDA(cudaMemcpyAsync(logits_out + (int64_t)i * V, S->logits + (int64_t)want[i] * S->logits_pitch, (size_t)V * 4, cudaMemcpyDeviceToHost,
                               ctx->stream));
    LMB_CUDA(cudaStreamSynchronize(ctx->stream));
    return check_device_error(ctx);
  }
  LMB_TRY(ensure_rows(S, Z.prompt, T, n_want));
  RowsBuf& r = Z.prompt;
  std::vector<int> meta((size_t)4 * T + 3 * B + n_want);
  RowsRun run;
  run.T = T; run.max_len = max_len; run.ctx_len = ctx_len;
  int at = 0;
  for (int b = 0; b < B; ++b) {
    run.h_start.push_back(at); run.h_len.push_back(lengths[b]); run.h_pos0.push_back(S->host_pos_v[b]);
    meta[(size_t)4 * T + b] = at; meta[(size_t)4 * T + B + b] = lengths[b]; meta[(size_t)4 * T + 2 * B + b] = S->host_pos_v[b];
    for (int i = 0; i < lengths[b]; ++i, ++at) {
      meta[at] = tokens[at];
      meta[(size_t)T + at] = b;
      meta[(size_t)2 * T + at] = S->host_pos_v[b] + i;
      meta[(size_t)3 * T + at] = i == lengths[b] - 1 ? b : -1;
    }
  }
  for (int i = 0; i < n_want; ++i) meta[(size_t)4 * T + 3 * B + i] = want[i];
  LMB_CUDA(cudaMemcpyAsync(r.meta, meta.data(), meta.size() * 4, cudaMemcpyHostToDevice, ctx->stream));
  run.tokens = r.meta; run.seq = r.meta + T; run.pos = r.meta + 2 * (int64_t)T; run.last = r.meta + 3 * (int64_t)T;
  run.start = r.meta + 4 * (int64_t)T; run.len = run.start + B; run.pos0 = run.len + B;
  const int* want_dev = run.pos0 + B;
  int32_t rc = rows_step(S, r, run, false, ctx->stream);
  if (rc == LMB200_OK && n_want > 0) {
    const bool to_session = greedy && n_want == B;
    rc = ensure_want(S, n_want);
    float* logits = to_session ? S->logits : Z.want_logits;
    const int pitch = to_session ? S->logits_pitch : V;
    if (rc == LMB200_OK) rc = rows_head(S, r, run, want_dev, n_want, Z.want_xn, logits, pitch, ctx->stream);
    if (rc == LMB200_OK && to_session) rc = argmax_launch(S, ctx->stream);
    if (rc == LMB200_OK && logits_out &&
        cudaMemcpy2DAsync(logits_out, (size_t)V * 4, logits, (size_t)pitch * 4, (size_t)V * 4, (size_t)n_want, cudaMemcpyDeviceToHost, ctx->stream) !=
            cudaSuccess)
      rc = fail(LMB200_ECUDA, "extend: logits copy failed");
  }
  const cudaError_t e = cudaStreamSynchronize(ctx->stream);       // also: `meta` is host memory of this call
  LMB_TRY(rc);
  if (e != cudaSuccess) return fail(LMB200_ECUDA, "extend: %s", cudaGetErrorString(e));
  for (int b = 0; b < B; ++b) S->host_pos_v[b] += lengths[b];
  LMB_TRY(push_positions(S));
  return check_device_error(ctx);
}

// bytes a decode step has to move: every weight once, latent rows (or the window's keys and values) of T positions per sequence (once
// for all heads, again for each layer that borrows them), recurrent states read and written, convolution inputs
int64_t layered_step_bytes(const Session* S, int32_t T) {
  const Model* M = S->m;
  const int64_t e = M->esz, W = M->cfg.hidden, B = S->B;
  int64_t n = (int64_t)M->cfg.vocab * W * e + W * 4 + B * W * e;
  for (int l = 0; l < M->cfg.n_layers; ++l) {
    const LayerSpec& s = M->specs[l];
    auto mat = [&](const WMap& m) { int64_t k = 0; for (int i = 0; i < kMaxSrc; ++i) k += (int64_t)m.src_rows[i] * m.src_cols[i]; return k * e; };
    n += mat(s.m_in) + mat(s.m_out) + W * 4;
    if (post_norm(M)) n += mat(s.m_gu) + mat(s.m_down) + mat(s.m_sg) + mat(s.m_sp) + mat(s.m_lr) + 2 * W * 4 + B * M->side_dim * e;
    if (is_attention(s)) n += B * (int64_t)((s.c.window > 0 ? std::min(T, s.c.window) : T) + (s.c.kv_from < 0 ? 1 : 0)) * s.c.kv_heads * (s.c.dim + s.c.vdim) * e;
    else if (is_latent(s)) n += mat(s.m_uq) + mat(s.m_ukv) + B * (int64_t)(T + (s.c.kv_from < 0 ? 1 : 0)) * (s.c.kv_rank + s.c.rot_dim) * e;
    else n += 2 * B * (int64_t)s.c.heads * s.c.dim * s.c.vdim * 4;
    if (is_delta(s)) n += B * (int64_t)delta_channels(s) * s.c.conv * 4;
  }
  return n;
}

int32_t layered_configure() {
  LMB_TRY(latent_configure());
  LMB_TRY(window_configure());
  LMB_TRY(delta_configure());
  return retention_configure();
}

}  // namespace lmb

using namespace lmb;

extern "C" int32_t lmb200_model_create_layered(lmb200_ctx hctx, const lmb200_layered_config* cfg, const lmb200_layer_config* layers,
                                               lmb200_model* out) {
  Ctx* ctx = ctx_from(hctx);
  if (!ctx) return LMB200_EINVAL;
  LMB_REQUIRE(cfg && layers && out, "model_create_layered: null argument");
  LMB_REQUIRE(cfg->n_layers >= 1 && cfg->width >= 1 && cfg->vocab >= 1, "model_create_layered: non-positive size");
  LMB_REQUIRE(cfg->width <= 12288, "model_create_layered: width %d (at most 12288)", cfg->width);
  LMB_REQUIRE(cfg->dtype == LMB200_F32 || cfg->dtype == LMB200_BF16, "model_create_layered: dtype %d", cfg->dtype);
  LMB_REQUIRE(cfg->softcap >= 0.f && cfg->eps >= 0.f, "model_create_layered: softcap %g, eps %g", cfg->softcap, cfg->eps);
  const int block = cfg->block;
  LMB_REQUIRE(block == LMB200_BLOCK_PARALLEL || block == LMB200_BLOCK_POSTNORM, "model_create_layered: block %d", block);
  LMB_REQUIRE(cfg->side_dim >= 0 && (block == LMB200_BLOCK_POSTNORM || (cfg->side_dim == 0 && !cfg->tied_head && (cfg->embed_scale == 0.f || cfg->embed_scale == 1.f))),
              "model_create_layered: token input of %d, tied head %d, embedding scale %g", cfg->side_dim, cfg->tied_head, cfg->embed_scale);
  std::vector<LayerSpec> specs;
  for (int l = 0; l < cfg->n_layers; ++l) {
    LMB_TRY(check_layer(layers[l], specs, l, block));
    LayerSpec s;
    s.c = layers[l];
    if (s.c.mixer == LMB200_MIXER_RETENTION || s.c.mixer == LMB200_MIXER_LIGHTNING) s.decay.assign(layers[l].decay, layers[l].decay + s.c.heads);
    if (has_state(s)) s.c.kv_from = -1;
    if (!is_latent(s)) s.c.q_rank = s.c.kv_rank = s.c.rot_dim = 0;
    if (is_delta(s)) s.c.rot_dims = 0;
    if (s.c.kv_heads == 0) s.c.kv_heads = s.c.heads;
    s.c.decay = nullptr;
    if (s.c.kv_from < 0) s.c.kv_from = -1;
    derive_layer(s, cfg->width, block, cfg->side_dim);
    specs.push_back(s);
  }
  LMB_CUDA(cudaSetDevice(ctx->device));
  Model* M = new Model();
  M->ctx = ctx;
  lmb200_model_config& c = M->cfg;
  c.n_layers = cfg->n_layers; c.hidden = cfg->width; c.vocab = cfg->vocab; c.rms_eps = cfg->eps; c.dtype = cfg->dtype;
  c.tp_size = 1; c.arch = LMB200_ARCH_LAYERED;
  M->esz = c.dtype == LMB200_BF16 ? 2 : 4;
  M->softcap = cfg->softcap;
  M->block = block; M->side_dim = cfg->side_dim; M->tied_head = cfg->tied_head != 0; M->embed_scale = cfg->embed_scale != 0.f ? cfg->embed_scale : 1.f;
  M->specs = specs;
  M->lw.resize(c.n_layers);
  M->m_head.kind = MAP_PLAIN;
  M->m_head.rows = c.vocab; M->m_head.K = c.hidden; M->m_head.src_rows[0] = c.vocab; M->m_head.src_cols[0] = c.hidden;
  finish_map(M->m_head);
  int32_t rc = LMB200_OK;
  auto alloc = [&](void** p, int64_t bytes) {
    if (rc != LMB200_OK) return;
    rc = dmalloc(p, bytes, true, ctx->stream);
    if (rc == LMB200_OK) M->weight_bytes += bytes;
  };
  auto upload = [&](float** p, const std::vector<float>& h) {
    alloc((void**)p, (int64_t)h.size() * 4);
    if (rc == LMB200_OK && !h.empty() && (cudaMemcpyAsync(*p, h.data(), h.size() * 4, cudaMemcpyHostToDevice, ctx->stream) != cudaSuccess ||
                                          cudaStreamSynchronize(ctx->stream) != cudaSuccess))
      rc = fail(LMB200_ECUDA, "model_create_layered: upload failed");
  };
  for (int l = 0; l < c.n_layers; ++l) {
    const LayerSpec& s = M->specs[l];
    LayeredWeights& w = M->lw[l];
    alloc(&w.w_in, tiled_elems(s.m_in, c.dtype) * M->esz);
    alloc(&w.w_out, tiled_elems(s.m_out, c.dtype) * M->esz);
    alloc((void**)&w.norm, (int64_t)c.hidden * 4);
    if (block == LMB200_BLOCK_POSTNORM) {
      if (s.c.ff) {
        alloc(&w.w_gu, tiled_elems(s.m_gu, c.dtype) * M->esz);
        alloc(&w.w_down, tiled_elems(s.m_down, c.dtype) * M->esz);
        alloc((void**)&w.norm2, (int64_t)c.hidden * 4);
      }
      if (M->side_dim) {
        alloc(&w.w_sg, tiled_elems(s.m_sg, c.dtype) * M->esz);
        alloc(&w.w_sp, tiled_elems(s.m_sp, c.dtype) * M->esz);
        alloc((void**)&w.side_norm, (int64_t)c.hidden * 4);
      }
    }
    const std::vector<float> f = rotation_freqs(s.c);
    upload(&w.inv_freq, f);
    if (!f.empty()) {
      size_t id = 0;
      while (id < M->rot_freqs.size() && M->rot_freqs[id] != f) ++id;
      if (id == M->rot_freqs.size()) M->rot_freqs.push_back(f);
      w.rot_id = (int)id;
    }
    if (is_latent(s)) {
      alloc(&w.w_uq, tiled_elems(s.m_uq, c.dtype) * M->esz);
      alloc(&w.w_ukv, tiled_elems(s.m_ukv, c.dtype) * M->esz);
      alloc(&w.w_ukt, (int64_t)s.c.heads * s.c.dim * s.c.kv_rank * M->esz);
      alloc(&w.w_uv, (int64_t)s.c.heads * s.c.vdim * s.c.kv_rank * M->esz);
      alloc((void**)&w.q_norm, (int64_t)s.c.q_rank * 4);
      if (s.c.kv_from < 0) alloc((void**)&w.kv_norm, (int64_t)s.c.kv_rank * 4);
    } else if (is_delta(s)) {
      alloc(&w.w_lr, tiled_elems(s.m_lr, c.dtype) * M->esz);
      alloc((void**)&w.conv, (int64_t)delta_channels(s) * s.c.conv * 4);
      alloc((void**)&w.a_log, (int64_t)s.c.heads * 4);
      alloc((void**)&w.dt_bias, (int64_t)s.c.heads * s.c.dim * 4);
      alloc((void**)&w.mix_norm, (int64_t)s.c.vdim * 4);
    } else if (!is_attention(s)) {
      if (is_lightning(s)) alloc((void**)&w.mix_norm, (int64_t)out_width(s) * 4);
      std::vector<float> d((size_t)s.c.heads * kDecayPow);
      for (int h = 0; h < s.c.heads; ++h)
        for (int i = 0; i < kDecayPow; ++i) d[(size_t)h * kDecayPow + i] = (float)pow(s.decay[h], i);
      upload(&w.decay, d);
    }
  }
  alloc(&M->embed, (int64_t)c.vocab * c.hidden * M->esz);
  alloc((void**)&M->final_norm, (int64_t)c.hidden * 4);
  if (M->side_dim) alloc(&M->side_embed, (int64_t)c.vocab * c.n_layers * M->side_dim * M->esz);
  alloc(&M->lm_head, tiled_elems(M->m_head, c.dtype) * M->esz);
  if (rc == LMB200_OK && cudaStreamSynchronize(ctx->stream) != cudaSuccess) rc = fail(LMB200_ECUDA, "model_create_layered: sync failed");
  if (rc != LMB200_OK) { lmb200_model_destroy(reinterpret_cast<lmb200_model>(M)); return rc; }
  *out = reinterpret_cast<lmb200_model>(M);
  return LMB200_OK;
}
