// Host-side launchers of the sequence-model mechanisms: RMS norms of a float32 residual stream, gated
// feed-forwards, recurrences (mLSTM, key-decayed matrix states) and attention (latent, grouped heads) over prompt portions
// and single tokens. Every size and constant
// is a parameter; the engine in core/seqmodel.cc strings them together, the C ABI also exposes them one by one.
//
// Rows: a step carries R = n_seq * T tokens, row r = s * T + t being token t of sequence s. Buffers named x are the
// float32 residual stream, dense [R, width]; all other activations are of the storage type T with a row pitch.
#pragma once
#include "kernels.h"

namespace ag { namespace k {

inline int64_t pad8(int64_t n) { return (n + 7) / 8 * 8; }

// ── norms and the feed-forward activation (rms_glu.cu) ──────────────────────
// x <- (load_x ? x : 0) + embed_scale embed[tok] (if embed) + rms(post) * post_w (if post) + step (if step), written back when anything was added or !load_x; then
// out1 = rms(x) * w1 and, if out2, out2 = rms(x) * w2 (float32 weights, results in the storage type). out1 may be null
// (the stream is only prepared).
struct RmsRowsDesc {
  DType dtype;                       // of embed, out1, out2
  float* x; int64_t rows; int width;
  bool load_x = true;
  const int32_t* tok = nullptr; const void* embed = nullptr; int64_t embed_ld = 0; int vocab = 0;
  float embed_scale = 1.f;
  const float* step = nullptr;
  const float* post = nullptr; const float* post_w = nullptr;   // dense [rows, width]: a sublayer's output, normed on its way into the stream
  const float* w1 = nullptr; void* out1 = nullptr; int64_t ld1 = 0;
  const float* w2 = nullptr; void* out2 = nullptr; int64_t ld2 = 0;
  const int32_t* row_map = nullptr;  // out row r takes x row row_map[r] (gathers the rows a head needs, post included); x is then not written
  float eps = 1e-5f;
};
Status rms_rows(cudaStream_t s, const RmsRowsDesc& d);
// out[r, 0 .. ff) = the gated activation of gu's columns, which come in
// blocks of `block` gates followed by the values they gate (block = ff: two halves; kGluBlock: as the GEMM's gated epilogue
// wants its weight rows).
constexpr int kGluBlock = 16;
inline int64_t glu_rows(int64_t ff) { return (ff + kGluBlock - 1) / kGluBlock * 2 * kGluBlock; }
Status glu(cudaStream_t s, DType dt, const void* gu, int64_t ld_in, void* out, int64_t ld_out, int64_t rows, int ff, int block, Glu kind, float limit);

// ── linears of a step with at most 16 rows (seq_skinny.cu) ──────────────────
// One launch runs up to kSeqSegs products against K-major weights [n, ld] (rows of length k). 16-bit models hand each product
// its stored input rows `a` (tensor cores); any model can hand all of them the float32 stream x, normalised on the way into shared
// memory as rms(x) * norm_w, or one stored input (CUDA cores).
enum class SeqOut : int { Store = 0, StoreF32 = 1, Glu = 2, AddF32 = 3 };
struct SeqSeg {
  const void* w = nullptr; int64_t ld = 0; int n = 0;      // Glu: n results from glu_rows(n) weight rows in blocks of kGluBlock gates | values
  const float* norm_w = nullptr;
  const void* a = nullptr; int64_t a_ld = 0;
  SeqOut mode = SeqOut::Store; k::Glu glu = k::Glu::Clamped; float limit = 0.f;
  void* out = nullptr; int64_t out_ld = 0;
};
constexpr int kSeqSegs = 3;
constexpr int kSeqSkinnyRows = 16;
struct SeqSkinnyDesc {
  DType dtype;
  int rows; int k;                                         // k: input length; weights are padded with zeros to pad8(k)
  const float* x = nullptr; float eps = 1e-5f;             // normalised input, dense [rows, k]
  const void* a = nullptr; int64_t a_ld = 0;               // or a stored one
  SeqSeg seg[kSeqSegs]; int n_seg = 0;
};
Status seq_skinny(cudaStream_t s, const SeqSkinnyDesc& d);
bool seq_skinny_fits(int64_t k);

// ── mLSTM (mlstm.cu) ────────────────────────────────────────────────────────
// proj rows: q (heads * dim) | k (heads * dim) | v (heads * vdim) | g (heads * vdim); gates rows (float32): i | f, `heads`
// each, without bias. State per sequence (float32): S [heads, dim, vdim], n [heads, dim], m [heads], in this order
// (mlstm_state_floats each). y rows receive o / rms(o) * norm * sigmoid(g).
struct MlstmDesc {
  DType dtype;
  int n_seq, T, heads, dim, vdim;
  float gate_cap, eps;
  const void* proj; int64_t ld;
  const float* gates; int64_t gates_ld;
  const float* gate_bias;            // [2 * heads]
  const float* norm;                 // [heads * vdim]
  float* state; int64_t state_stride;  // floats between sequences
  void* y; int64_t y_ld;
  void* work = nullptr;              // mlstm_prefill only: mlstm_work_bytes
  bool simple = false;               // keeps 16-bit portions on the CUDA-core kernels
};
inline int64_t mlstm_state_floats(int heads, int dim, int vdim) { return ((int64_t)heads * ((int64_t)dim * vdim + dim + 1) + 3) / 4 * 4; }
size_t mlstm_work_bytes(int n_seq, int T, int heads, int dim, int vdim);
Status mlstm_prefill(cudaStream_t s, const MlstmDesc& d);   // chunk-parallel, any T
Status mlstm_step(cudaStream_t s, const MlstmDesc& d);      // token by token, for short portions

// ── latent attention (latent_attention.cu) ──────────────────────────────────
// proj rows: q head by head (dim | rot_dim), then the latent (kv_rank) and the shared rotated key part (rot_dim).
// Cache row of a token: latent at column 0, rotated key part at column pad8(kv_rank); pitch latent_cache_ld.
// rot_table: float2 (cos, sin), amplitude included, [max positions, rot_pairs].
struct LatentDesc {
  DType dtype;
  int n_seq, T, heads, dim, rot_dim, vdim, kv_rank, rot_pairs;
  float scale, eps;
  void* proj; int64_t ld;
  const float* c_norm;               // [kv_rank]
  const float2* rot_table;
  void* cache; int64_t seq_stride;   // elements between sequences' caches
  const int* pos;                    // device: tokens already cached, per sequence
  int max_len;
  const void* w_uk; const void* w_uv; int64_t w_ld;   // [heads * dim, kv_rank], [heads * vdim, kv_rank]
  void* y; int64_t y_ld;
};
inline int64_t latent_cache_ld(int kv_rank, int rot_dim) { return pad8(kv_rank) + pad8(rot_dim); }
// Rotates q in place, norms the latent, rotates the key part and appends both to the cache (rows pos .. pos + T).
Status latent_append(cudaStream_t s, const LatentDesc& d);
// Short portions attend in the latent space (the up-projections absorbed into query and output); longer ones expand keys and
// values per head and take prompt_attention.
// work: latent_decode_work_bytes.
size_t latent_decode_work_bytes(int rows, int heads, int kv_rank, int rot_dim, int max_len);
Status latent_decode(cudaStream_t s, const LatentDesc& d, void* work);

// ── matrix states with one decay per key channel (key_decay.cu, key_decay_chunk.cuh) ──
// Per head S [dim, vdim], row d of which fades by a_d in every token:
//     S <- diag(a) S,   u = v, or with the delta rule beta (v - S^T k),   S <- S + k u^T,   o = S^T q.
// y rows receive o / rms(o) * norm * act(gate). Options, each on its own:
//   delta      the delta rule; beta = sigmoid(beta_raw), one per head
//   taps       > 0: q, k and v pass a causal convolution of that many taps per channel, then silu
//   unit       q and k become unit vectors per head, x / sqrt(|x|^2 + 1e-6)
//   softplus   a = exp(-rate_h softplus(z + bias)); otherwise a = sigmoid(z + bias)^(1 / tau)
//   gate_silu  silu instead of sigmoid on the gate
// proj row: q at column q_off (qk_heads * dim), k, v (heads * vdim), a1 (rank a_rank, z = a2 a1) and either the gate itself at
// g_off (g_rank 0) or g1 there (rank g_rank, gate = g2 g1). Head h uses q / k head h / (heads / qk_heads). q is multiplied by q_scale.
// Memory of a sequence: S of all heads (float32), then with taps the last raw q | k | v inputs as a ring of key_decay_ring rows
// of the storage type, row (position % ring) holding the token at that position.
constexpr int kKeyDecayStepTokens = 16;    // portions up to here go token by token in one launch
struct KeyDecayDesc {
  DType dtype;
  int n_seq, T, heads, qk_heads, dim, vdim;
  bool delta = false, unit = false, softplus = false, gate_silu = false;
  int taps = 0;
  float tau = 1.f, q_scale = 1.f, eps;
  const void* proj; int64_t ld;
  int q_off, k_off, v_off, a_off, a_rank, g_off, g_rank = 0;
  const void* a2; const void* g2 = nullptr;      // [heads * dim, pad8(a_rank)], [heads * vdim, pad8(g_rank)], storage type
  const float* bias; const float* rate = nullptr; const float* conv = nullptr; const float* norm;   // [heads * dim], [heads], [channels, taps], [vdim]
  const float* beta = nullptr; int64_t beta_ld = 0;
  void* mem; int64_t mem_stride;                 // bytes between sequences
  const int* pos;                                // device: tokens already taken in, per sequence
  void* y; int64_t y_ld;
  void* work = nullptr;                          // key_decay_work_bytes
  bool simple = false;                           // keeps 16-bit portions on the token-by-token kernel
};
inline int key_decay_channels(int heads, int qk_heads, int dim, int vdim) { return 2 * qk_heads * dim + heads * vdim; }
inline int key_decay_ring(int taps) { return taps > 1 ? taps - 1 + kKeyDecayStepTokens : 0; }
inline size_t key_decay_state_bytes(int heads, int dim, int vdim) { return ((size_t)heads * dim * vdim * sizeof(float) + 15) / 16 * 16; }
inline size_t key_decay_mem_bytes(DType dt, int heads, int qk_heads, int dim, int vdim, int taps) {
  return key_decay_state_bytes(heads, dim, vdim) + ((size_t)key_decay_ring(taps) * key_decay_channels(heads, qk_heads, dim, vdim) * dtype_size(dt) + 15) / 16 * 16;
}
size_t key_decay_work_bytes(const KeyDecayDesc& d);
Status key_decay(cudaStream_t s, const KeyDecayDesc& d, int* launches);      // picks the forms below by T, dtype and sizes
bool key_decay_chunk_eligible(const KeyDecayDesc& d);                        // 16-bit portions in chunks, tensor cores

// ── attention of heads that share keys in groups (grouped_attention.cu) ─────
// proj row: q (heads * dim), then, unless `shared`, k (kv_heads * dim) and v (kv_heads * vdim), at the given columns. Cache row of a
// token: keys, then values at column pad8(kv_heads * dim); pitch grouped_cache_ld. Queries and keys are normed per head
// (x / rms(x) * weight) and their first 2 * rot_pairs entries turned, entry i with entry i + rot_pairs. `shared`: keys and
// values are another layer's, already in the cache.
struct GroupedAttnDesc {
  DType dtype;
  int n_seq, T, heads, kv_heads, dim, vdim, rot_pairs, window = 0;
  bool shared = false;
  float scale, softcap = 0.f, eps;
  void* proj; int64_t ld;
  int q_off = 0, k_off = 0, v_off = 0;
  const float* q_norm; const float* k_norm = nullptr;
  const float2* rot_table;               // (cos, sin), amplitude included, [max positions, rot_pairs]
  void* cache; int64_t seq_stride;       // elements between sequences' caches
  const int* pos; int max_len;           // device: tokens already cached, per sequence (before this step, also when `shared`)
  void* y; int64_t y_ld;
};
inline int64_t grouped_v_col(int kv_heads, int dim) { return pad8((int64_t)kv_heads * dim); }
inline int64_t grouped_cache_ld(int kv_heads, int dim, int vdim) { return grouped_v_col(kv_heads, dim) + pad8((int64_t)kv_heads * vdim); }
Status grouped_append(cudaStream_t s, const GroupedAttnDesc& d);             // norms and turns q in place, writes cache rows pos .. pos + T
Status grouped_decode(cudaStream_t s, const GroupedAttnDesc& d);             // short portions; grouped_append comes first

// ── attention of a prompt portion (prompt_attention.cu, prompt_attention_tc.cu) ──
// T new rows per sequence over past + T rows of keys and values. A query row holds `heads` x (dim | rot_dim); `group` neighbouring
// heads share one key head of k (dim each) and v (vdim each); the rot_dim entries meet k_rot, which all heads share. Row t of
// the portion sees the keys up to past + t, the last `window` of them (0: all). softcap c > 0: scores become c tanh(score / c).
// The *_b strides step from sequence to sequence.
struct PromptAttnDesc {
  DType dtype;
  int n_seq = 1, T, past, heads, group = 1, dim, rot_dim = 0, vdim, window = 0;
  float scale, softcap = 0.f;
  const void* q; int64_t q_ld;
  const void* k; int64_t k_ld;
  const void* v; int64_t v_ld;
  const void* k_rot = nullptr; int64_t k_rot_ld = 0;
  void* y; int64_t y_ld;
  int64_t q_b = 0, k_b = 0, v_b = 0, k_rot_b = 0, y_b = 0;
};
Status prompt_attention(cudaStream_t s, const PromptAttnDesc& d);       // picks one of the two below
bool prompt_attention_tc_eligible(const PromptAttnDesc& d);             // 16-bit, tensor cores
Status prompt_attention_tc(cudaStream_t s, const PromptAttnDesc& d);

// ── bookkeeping of a step (seq_skinny.cu) ───────────────────────────────────
// pos[s] += T for every sequence; with `history`: tokens also go to history[*step][s] and *step advances.
Status seq_advance(cudaStream_t s, int* pos, int n_seq, int T, const int32_t* tok, int32_t* history, int* step, int max_steps);

}}  // namespace ag::k
