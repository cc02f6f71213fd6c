// Host-side launchers of the sequence-model mechanisms: RMS norms of a float32 residual stream, the clamped gated
// feed-forward, the mLSTM recurrence and latent attention (prompt portions and single tokens). Every size and constant
// is a parameter; the engine in core/seqmodel.cc strings them together, the C ABI also exposes them one by one.
//
// Rows: a step carries R = n_seq * T tokens, row r = s * T + t being token t of sequence s. Buffers named x are the
// float32 residual stream, dense [R, width]; all other activations are of the storage type T with a row pitch.
#pragma once
#include "kernels.h"

namespace ag { namespace k {

inline int64_t pad8(int64_t n) { return (n + 7) / 8 * 8; }

// ── norms and the feed-forward activation (rms_glu.cu) ──────────────────────
// x <- (load_x ? x : 0) + embed[tok] (if embed) + step (if step), written back when anything was added or !load_x; then
// out1 = rms(x) * w1 and, if out2, out2 = rms(x) * w2 (float32 weights, results in the storage type). out1 may be null
// (the stream is only prepared).
struct RmsRowsDesc {
  DType dtype;                       // of embed, out1, out2
  float* x; int64_t rows; int width;
  bool load_x = true;
  const int32_t* tok = nullptr; const void* embed = nullptr; int64_t embed_ld = 0; int vocab = 0;
  const float* step = nullptr;
  const float* w1 = nullptr; void* out1 = nullptr; int64_t ld1 = 0;
  const float* w2 = nullptr; void* out2 = nullptr; int64_t ld2 = 0;
  const int32_t* row_map = nullptr;  // out row r takes x row row_map[r] (gathers the rows a head needs); x is then not written
  float eps = 1e-5f;
};
Status rms_rows(cudaStream_t s, const RmsRowsDesc& d);
// out[r, 0 .. ff) = g sigmoid(1.702 g) (u + 1), g = min(gate, limit), u = clamp(up, -limit, limit); the columns of gu come in
// blocks of `block` gates followed by the values they gate (block = ff: two halves; kGluBlock: as the GEMM's gated epilogue
// wants its weight rows).
constexpr int kGluBlock = 16;
inline int64_t glu_rows(int64_t ff) { return (ff + kGluBlock - 1) / kGluBlock * 2 * kGluBlock; }
Status clamped_glu(cudaStream_t s, DType dt, const void* gu, int64_t ld_in, void* out, int64_t ld_out, int64_t rows, int ff, int block, float limit);

// ── linears of a step with at most 16 rows (seq_skinny.cu) ──────────────────
// One launch runs up to kSeqSegs products against K-major weights [n, ld] (rows of length k). 16-bit models hand each product
// its stored input rows `a` (tensor cores); any model can hand all of them the float32 stream x, normalised on the way into shared
// memory as rms(x) * norm_w, or one stored input (CUDA cores).
enum class SeqOut : int { Store = 0, StoreF32 = 1, Glu = 2, AddF32 = 3 };
struct SeqSeg {
  const void* w = nullptr; int64_t ld = 0; int n = 0;      // Glu: n results from glu_rows(n) weight rows in blocks of kGluBlock gates | values
  const float* norm_w = nullptr;
  const void* a = nullptr; int64_t a_ld = 0;
  SeqOut mode = SeqOut::Store; float limit = 0.f;
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
// Attention of T new rows per sequence over past + T cached rows, with keys and values expanded per head: kv rows
// [past + T, kv_ld] hold k (heads * dim) | v at column v_off (heads * vdim). The *_b strides step from sequence to sequence.
struct LatentPrefillDesc {
  DType dtype;
  int n_seq = 1, T, past, heads, dim, rot_dim, vdim;
  float scale;
  const void* q; int64_t q_ld;
  const void* kv; int64_t kv_ld; int64_t v_off;
  const void* k_rot; int64_t k_rot_ld;
  void* y; int64_t y_ld;
  int64_t q_b = 0, kv_b = 0, k_rot_b = 0, y_b = 0;
};
Status latent_prefill(cudaStream_t s, const LatentPrefillDesc& d);      // picks one of the two below
bool latent_prefill_tc_eligible(const LatentPrefillDesc& d);            // 16-bit, tensor cores (latent_attention_tc.cu)
Status latent_prefill_tc(cudaStream_t s, const LatentPrefillDesc& d);
// The same for short portions, attending in the latent space (the up-projections absorbed into query and output).
// work: latent_decode_work_bytes.
size_t latent_decode_work_bytes(int rows, int heads, int kv_rank, int rot_dim, int max_len);
Status latent_decode(cudaStream_t s, const LatentDesc& d, void* work);

// ── bookkeeping of a step (seq_skinny.cu) ───────────────────────────────────
// pos[s] += T for every sequence; with `history`: tokens also go to history[*step][s] and *step advances.
Status seq_advance(cudaStream_t s, int* pos, int n_seq, int T, const int32_t* tok, int32_t* history, int* step, int max_steps);

}}  // namespace ag::k
