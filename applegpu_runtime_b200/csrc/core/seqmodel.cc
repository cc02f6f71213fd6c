// Engine of the sequence models: weights, per-sequence memory, prompt portions and generated tokens.
//
// A model is a list of layers over a float32 residual stream, in one of two forms:
//     parallel    x <- x + mixer(rms(x) w1) + ff(rms(x) w2)
//     sequential  x <- x + rms(mixer(rms(x) w1)) p1, then x <- x + rms(ff(rms(x) w2)) p2
// A range of layers may run several times with the same weights, every run with its own memory. What distinguishes the mixers
// (columns of their input product, memory, kernels) sits behind the Mixer interface below, so another design adds a mixer
// kind and keeps the rest.
//
// Memory: the engine owns `slots` sequences of at most `max_len` tokens. A layer run keeps, for every slot, a fixed block
// (recurrent state) or a row per token (cache); a layer may also use the cache of an earlier one. The number of tokens a slot holds lives in device memory (kernels read it
// there, so that a captured step serves every length) with a mirror on the host.
//
// A step brings the next T tokens of n consecutive slots (R = n T rows) and picks its kernels by size: up to 16 rows the
// linears stream their weights through seq_skinny, more go to the GEMM; up to 16 tokens a sequence the mixers run token by
// token, longer portions in their chunk-parallel / expanded form. A step with T = 1 is captured once per slot range as a
// CUDA graph that ends by picking each sequence's next token on the device; greedy generation replays it.
#include "seqmodel.h"
#include "../kernels/seq_kernels.h"
#include <atomic>
#include <algorithm>
#include <cmath>

namespace ag {

extern std::atomic<uint64_t> g_launch_count;
namespace profile { long begin(const std::string& name, double work); void end(long i); bool enabled(); }

namespace {

// One timed launch (or group of launches) of a step; work is flops for products and prompt attention, bytes otherwise.
struct Span {
  long i;
  Span(const char* name, double work) : i(profile::begin(name, work)) {}
  ~Span() { profile::end(i); }
};
double product(double m, double n, double kdim) { return 2.0 * m * n * kdim; }

constexpr int kShortT = 16;             // tokens per sequence up to which mixers run token by token
constexpr int kMaxRows = 8192;          // rows of a step; longer portions are cut
using k::pad8;

struct Scratch {                        // a device buffer that grows
  std::shared_ptr<Buffer> buf;
  void* ptr() const { return buf ? buf->ptr : nullptr; }
};

struct SeqEngine;

// What a step hands to a mixer.
struct StepCtx {
  cudaStream_t s;
  int slot0, n_seq, T;
  const int* host_len;                  // tokens held by slot0 .. before this step
  int rows() const { return n_seq * T; }
};

// A token mixer of one layer: sizes, memory, kernels. proj is the input product of the step (storage type, pitch ld), y
// receives heads * vdim columns that the layer's output product reads.
struct Mixer {
  const SeqLayerCfg& c;
  const TensorRec* w;                   // kSeqLayerWeights records
  DType dtype;
  Mixer(const SeqLayerCfg& cfg, const TensorRec* weights, DType dt) : c(cfg), w(weights), dtype(dt) {}
  virtual ~Mixer() {}
  virtual int proj_cols() const = 0;
  virtual int gate_cols() const { return 0; }        // float32 projections (kWAux0)
  virtual size_t slot_bytes(int max_len) const = 0;
  virtual bool clear_on_reset() const = 0;
  virtual Status check(const SeqModelCfg& m, int max_len) const = 0;
  virtual size_t kv_bytes(const int*, int, int) const { return 0; }   // expanded keys and values of a step
  virtual size_t work_bytes(int n_seq, int T, int max_len) const = 0;
  virtual Status run(const StepCtx& x, void* proj, int64_t ld, const float* gates, void* mem, int max_len, const int* pos, void* y, int64_t y_ld, void* work, void* kv,
                     float eps, int* launches) const = 0;
};

bool is_matrix(const TensorRec& t, DType dt, int64_t rows, int64_t cols) {
  return t.buf && t.contiguous() && t.dtype == dt && t.shape.size() == 2 && t.shape[0] == rows && t.shape[1] == cols;
}
bool is_vector(const TensorRec& t, int64_t n) { return t.buf && t.contiguous() && t.dtype == DType::F32 && numel_of(t.shape) == n; }
const float* f32(const TensorRec& t) { return static_cast<const float*>(t.data()); }

k::GemmDesc linear_desc(DType dt, const void* a, int64_t a_ld, int64_t m, int64_t kdim, const void* w, int64_t w_ld, int64_t n, void* out, int64_t out_ld, bool out_f32,
                        const float* residual) {
  k::GemmDesc g;
  g.dtype = dt; g.b_dtype = dt; g.a = a; g.b = w; g.c = out; g.m = m; g.n = n; g.k = kdim; g.batch = 1;
  g.a_row = a_ld; g.a_col = 1; g.a_batch = 0; g.b_row = 1; g.b_col = w_ld; g.b_batch = 0; g.c_row = out_ld; g.c_batch = 0;
  g.c_f32 = out_f32 && dt != DType::F32;
  g.ep.residual = residual;
  return g;
}

// ── mixers ──────────────────────────────────────────────────────────────────
struct MlstmMixer : Mixer {
  using Mixer::Mixer;
  int proj_cols() const override { return 2 * c.heads * (c.dim + c.vdim); }
  int gate_cols() const override { return 2 * c.heads; }
  size_t slot_bytes(int) const override { return (size_t)k::mlstm_state_floats(c.heads, c.dim, c.vdim) * sizeof(float); }
  bool clear_on_reset() const override { return true; }
  Status check(const SeqModelCfg& m, int) const override {
    if (!is_matrix(w[kWAux0], dtype, 2 * c.heads, pad8(m.width)) || !is_vector(w[kWAux1], 2 * c.heads) || !is_vector(w[kWAux2], (int64_t)c.heads * c.vdim))
      return Status::invalid("mLSTM gate weights, gate bias or head norm");
    if (!(c.gate_cap > 0.f)) return Status::invalid("mLSTM gate cap must be positive");
    return Status::OK();
  }
  size_t work_bytes(int n_seq, int T, int) const override { return T <= kShortT ? 0 : k::mlstm_work_bytes(n_seq, T, c.heads, c.dim, c.vdim); }
  Status run(const StepCtx& x, void* proj, int64_t ld, const float* gates, void* mem, int max_len, const int*, void* y, int64_t y_ld, void* work, void*, float eps,
             int* launches) const override {
    k::MlstmDesc d;
    d.dtype = dtype; d.n_seq = x.n_seq; d.T = x.T; d.heads = c.heads; d.dim = c.dim; d.vdim = c.vdim; d.gate_cap = c.gate_cap; d.eps = eps;
    d.proj = proj; d.ld = ld; d.gates = gates; d.gates_ld = gate_cols(); d.gate_bias = f32(w[kWAux1]); d.norm = f32(w[kWAux2]);
    d.state_stride = (int64_t)(slot_bytes(max_len) / sizeof(float));
    d.state = static_cast<float*>(mem) + x.slot0 * d.state_stride;
    d.y = y; d.y_ld = y_ld; d.work = work;
    const double row = (2.0 * c.dim + 3.0 * c.vdim) * dtype_size(dtype), mem_rw = 8.0 * c.dim * c.vdim;      // q k v g y; the state read and written once
    Span span(x.T <= kShortT ? "mlstm_step" : "mlstm_prefill", c.heads * (row * x.rows() + mem_rw * x.n_seq));
    if (x.T <= kShortT) { *launches += 1; return k::mlstm_step(x.s, d); }
    *launches += 4;
    return k::mlstm_prefill(x.s, d);
  }
};

struct LatentMixer : Mixer {
  using Mixer::Mixer;
  int proj_cols() const override { return c.heads * (c.dim + c.rot_dim) + c.kv_rank + c.rot_dim; }
  int64_t cld() const { return k::latent_cache_ld(c.kv_rank, c.rot_dim); }
  int64_t kv_cols() const { return pad8((int64_t)c.heads * c.dim) + pad8((int64_t)c.heads * c.vdim); }   // values start 16-byte aligned
  size_t slot_bytes(int max_len) const override { return (size_t)max_len * cld() * dtype_size(dtype); }
  bool clear_on_reset() const override { return false; }
  Status check(const SeqModelCfg&, int max_len) const override {
    if (c.kv_rank < 1 || c.kv_rank > 1024 || c.rot_dim < 0 || 2 * c.rot_pairs > c.rot_dim) return Status::invalid("latent attention sizes");
    if (!is_vector(w[kWAux0], c.kv_rank) || !is_matrix(w[kWAux1], dtype, kv_cols(), pad8(c.kv_rank))) return Status::invalid("latent norm or up-projections");
    if (c.rot_pairs && !(w[kWAux2].buf && w[kWAux2].contiguous() && w[kWAux2].dtype == DType::F32 && numel_of(w[kWAux2].shape) >= (int64_t)max_len * c.rot_pairs * 2))
      return Status::invalid("rotation table");
    return Status::OK();
  }
  size_t kv_bytes(const int* host_len, int n_seq, int T) const override {
    size_t worst = 0;
    for (int i = 0; i < n_seq;) {
      int n = 1;
      while (i + n < n_seq && host_len[i + n] == host_len[i]) n++;
      worst = std::max(worst, (size_t)n * (host_len[i] + T));
      i += n;
    }
    return worst * kv_cols() * dtype_size(dtype);
  }
  size_t work_bytes(int n_seq, int T, int max_len) const override {
    return T <= kShortT ? k::latent_decode_work_bytes(n_seq * T, c.heads, c.kv_rank, c.rot_dim, max_len) : 0;
  }
  Status run(const StepCtx& x, void* proj, int64_t ld, const float*, void* mem, int max_len, const int* pos, void* y, int64_t y_ld, void* work, void* kv, float eps,
             int* launches) const override {
    const size_t esz = dtype_size(dtype);
    k::LatentDesc d;
    d.dtype = dtype; d.n_seq = x.n_seq; d.T = x.T; d.heads = c.heads; d.dim = c.dim; d.rot_dim = c.rot_dim; d.vdim = c.vdim; d.kv_rank = c.kv_rank;
    d.rot_pairs = c.rot_pairs; d.scale = c.score_scale; d.eps = eps; d.proj = proj; d.ld = ld; d.c_norm = f32(w[kWAux0]);
    d.rot_table = reinterpret_cast<const float2*>(w[kWAux2].data());
    d.seq_stride = (int64_t)max_len * cld();
    d.cache = static_cast<uint8_t*>(mem) + (size_t)x.slot0 * slot_bytes(max_len);
    d.pos = pos; d.max_len = max_len;
    const uint8_t* wkv = static_cast<const uint8_t*>(w[kWAux1].data());
    const int64_t w_ld = pad8(c.kv_rank), v_off = pad8((int64_t)c.heads * c.dim);
    d.w_uk = wkv; d.w_uv = wkv + (size_t)v_off * w_ld * esz; d.w_ld = w_ld; d.y = y; d.y_ld = y_ld;
    if (x.T <= kShortT) {
      double keys = 0;
      for (int i = 0; i < x.n_seq; i++) keys += x.host_len[i] + x.T;
      Span span("latent_decode", esz * (keys * cld() + (double)c.heads * (c.dim + c.vdim) * c.kv_rank));
      *launches += 3;
      return k::latent_decode(x.s, d, work);
    }
    {
      Span span("latent_append", esz * (double)x.rows() * (2.0 * c.heads * c.rot_dim + 2.0 * (c.kv_rank + c.rot_dim)));
      AG_RETURN_IF_ERROR(k::latent_append(x.s, d));
    }
    *launches += 1;
    // sequences that hold equally many tokens share the two launches
    for (int i = 0; i < x.n_seq;) {
      int n = 1;
      while (i + n < x.n_seq && x.host_len[i + n] == x.host_len[i]) n++;
      const int past = x.host_len[i], keys = past + x.T;
      uint8_t* cache = static_cast<uint8_t*>(d.cache) + (size_t)i * slot_bytes(max_len);
      {
        Span span("latent_expand", n * product(keys, kv_cols(), c.kv_rank));
        k::GemmDesc g = linear_desc(dtype, cache, cld(), keys, c.kv_rank, wkv, w_ld, kv_cols(), kv, kv_cols(), false, nullptr);
        g.batch = n; g.a_batch = d.seq_stride; g.c_batch = keys * kv_cols();
        AG_RETURN_IF_ERROR(k::matmul(x.s, g));
      }
      k::PromptAttnDesc p;
      p.dtype = dtype; p.n_seq = n; p.T = x.T; p.past = past; p.heads = c.heads; p.dim = c.dim; p.rot_dim = c.rot_dim; p.vdim = c.vdim; p.scale = c.score_scale;
      p.q = static_cast<uint8_t*>(proj) + (size_t)i * x.T * ld * esz; p.q_ld = ld; p.q_b = x.T * ld;
      p.k = kv; p.k_ld = kv_cols(); p.v = static_cast<uint8_t*>(kv) + (size_t)v_off * esz; p.v_ld = kv_cols(); p.k_b = p.v_b = keys * kv_cols();
      p.k_rot = cache + (size_t)pad8(c.kv_rank) * esz; p.k_rot_ld = cld(); p.k_rot_b = d.seq_stride;
      p.y = static_cast<uint8_t*>(y) + (size_t)i * x.T * y_ld * esz; p.y_ld = y_ld; p.y_b = x.T * y_ld;
      Span span("latent_prefill", 2.0 * n * c.heads * (c.dim + c.rot_dim + c.vdim) * (past * (double)x.T + 0.5 * x.T * (x.T + 1.0)));
      AG_RETURN_IF_ERROR(k::prompt_attention(x.s, p));
      *launches += 2;
      i += n;
    }
    return Status::OK();
  }
};

// Matrix states with one decay per key channel: gated linear attention, the channel-wise gated delta rule.
struct KeyDecayMixer : Mixer {
  using Mixer::Mixer;
  bool delta() const { return c.flags & kKdDelta; }
  int qk_cols() const { return (int)pad8((int64_t)c.kv_heads * c.dim); }
  int v_cols() const { return (int)pad8((int64_t)c.heads * c.vdim); }
  int proj_cols() const override { return 2 * qk_cols() + v_cols() + (int)pad8(c.a_rank) + (c.g_rank ? (int)pad8(c.g_rank) : v_cols()); }
  int gate_cols() const override { return delta() ? c.heads : 0; }
  size_t slot_bytes(int) const override { return k::key_decay_mem_bytes(dtype, c.heads, c.kv_heads, c.dim, c.vdim, c.taps); }
  bool clear_on_reset() const override { return true; }
  Status check(const SeqModelCfg& m, int) const override {
    if (c.kv_heads < 1 || c.heads % c.kv_heads || c.a_rank < 1 || c.g_rank < 0 || c.taps < 0 || !(c.tau > 0.f)) return Status::invalid("key decay sizes");
    if (delta() && !is_matrix(w[kWAux0], dtype, c.heads, pad8(m.width))) return Status::invalid("write strengths");
    if (!is_matrix(w[kWAux1], dtype, (int64_t)c.heads * c.dim, pad8(c.a_rank)) || !is_vector(w[kWAux2], (int64_t)c.heads * c.dim) || !is_vector(w[kWAux3], c.vdim))
      return Status::invalid("decay weights, decay bias or head norm");
    if (c.g_rank && !is_matrix(w[kWAux4], dtype, (int64_t)c.heads * c.vdim, pad8(c.g_rank))) return Status::invalid("gate weights");
    if ((c.flags & kKdSoftplus) && !is_vector(w[kWAux5], c.heads)) return Status::invalid("decay rates");
    if (c.taps && !is_vector(w[kWAux6], (int64_t)k::key_decay_channels(c.heads, c.kv_heads, c.dim, c.vdim) * c.taps)) return Status::invalid("convolution taps");
    return Status::OK();
  }
  k::KeyDecayDesc desc(int n_seq, int T) const {
    k::KeyDecayDesc d;
    d.dtype = dtype; d.n_seq = n_seq; d.T = T; d.heads = c.heads; d.qk_heads = c.kv_heads; d.dim = c.dim; d.vdim = c.vdim;
    d.delta = delta(); d.unit = c.flags & kKdUnit; d.softplus = c.flags & kKdSoftplus; d.gate_silu = c.flags & kKdGateSilu;
    d.taps = c.taps; d.tau = c.tau; d.q_scale = (float)(1.0 / std::sqrt((double)c.dim));
    d.q_off = 0; d.k_off = qk_cols(); d.v_off = 2 * qk_cols(); d.a_off = d.v_off + v_cols(); d.a_rank = c.a_rank; d.g_off = d.a_off + (int)pad8(c.a_rank); d.g_rank = c.g_rank;
    return d;
  }
  size_t work_bytes(int n_seq, int T, int) const override { return k::key_decay_work_bytes(desc(n_seq, T)); }
  Status run(const StepCtx& x, void* proj, int64_t ld, const float* gates, void* mem, int max_len, const int* pos, void* y, int64_t y_ld, void* work, void*, float eps,
             int* launches) const override {
    k::KeyDecayDesc d = desc(x.n_seq, x.T);
    d.eps = eps; d.proj = proj; d.ld = ld; d.a2 = w[kWAux1].data(); d.bias = f32(w[kWAux2]); d.norm = f32(w[kWAux3]);
    if (c.g_rank) d.g2 = w[kWAux4].data();
    if (d.softplus) d.rate = f32(w[kWAux5]);
    if (c.taps) d.conv = f32(w[kWAux6]);
    d.beta = gates; d.beta_ld = gate_cols();
    d.mem_stride = (int64_t)slot_bytes(max_len);
    d.mem = static_cast<uint8_t*>(mem) + x.slot0 * d.mem_stride;
    d.pos = pos; d.y = y; d.y_ld = y_ld; d.work = work;
    const double esz = dtype_size(dtype), mem_rw = 8.0 * c.heads * c.dim * c.vdim;       // the state read and written once
    const double row = esz * (2.0 * c.kv_heads * c.dim + c.heads * c.vdim * (c.g_rank ? 2.0 : 3.0) + c.a_rank + c.g_rank), wts = esz * c.heads * ((double)c.dim * c.a_rank + (double)c.vdim * c.g_rank);
    const bool step = x.T <= k::kKeyDecayStepTokens;
    Span span(step ? (delta() ? "delta_step" : "gla_step") : delta() ? "delta_prefill" : "gla_prefill", row * x.rows() + mem_rw * x.n_seq + wts);
    return k::key_decay(x.s, d, launches);
  }
};

// Query heads in groups over shared keys and values, all of them or a window, with per-head norms and rotation.
struct GroupedMixer : Mixer {
  using Mixer::Mixer;
  bool shared() const { return c.kv_from >= 0; }
  int q_cols() const { return (int)pad8((int64_t)c.heads * c.dim); }
  int k_cols() const { return (int)pad8((int64_t)c.kv_heads * c.dim); }
  int proj_cols() const override { return q_cols() + (shared() ? 0 : k_cols() + (int)pad8((int64_t)c.kv_heads * c.vdim)); }
  int64_t cld() const { return k::grouped_cache_ld(c.kv_heads, c.dim, c.vdim); }
  size_t cache_bytes(int max_len) const { return (size_t)max_len * cld() * dtype_size(dtype); }
  size_t slot_bytes(int max_len) const override { return shared() ? 0 : cache_bytes(max_len); }
  bool clear_on_reset() const override { return false; }
  Status check(const SeqModelCfg& m, int max_len) const override {
    if (c.kv_heads < 1 || c.heads % c.kv_heads || c.window < 0 || 2 * c.rot_pairs > c.dim) return Status::invalid("grouped attention sizes");
    if (!is_vector(w[kWAux0], c.dim) || (!shared() && !is_vector(w[kWAux1], c.dim))) return Status::invalid("query or key norm");
    if (c.rot_pairs && !(w[kWAux2].buf && w[kWAux2].contiguous() && w[kWAux2].dtype == DType::F32 && numel_of(w[kWAux2].shape) >= (int64_t)max_len * c.rot_pairs * 2))
      return Status::invalid("rotation table");
    if (shared()) {
      if (c.kv_from >= (int)m.layers.size()) return Status::invalid("no such layer to take keys from");
      const SeqLayerCfg& o = m.layers[c.kv_from];
      if (o.mixer != MixerKind::GroupedAttention || o.kv_from >= 0 || o.kv_heads != c.kv_heads || o.dim != c.dim || o.vdim != c.vdim) return Status::invalid("the layer to take keys from has none of this kind");
    }
    return Status::OK();
  }
  size_t work_bytes(int, int, int) const override { return 0; }
  double pairs_seen(int past, int T) const {            // (query, key) pairs of a portion
    double n = 0;
    for (int t = 0; t < T; t++) n += c.window ? std::min(c.window, past + t + 1) : past + t + 1;
    return n;
  }
  Status run(const StepCtx& x, void* proj, int64_t ld, const float*, void* mem, int max_len, const int* pos, void* y, int64_t y_ld, void*, void*, float eps, int* launches) const override {
    const size_t esz = dtype_size(dtype);
    k::GroupedAttnDesc d;
    d.dtype = dtype; d.n_seq = x.n_seq; d.T = x.T; d.heads = c.heads; d.kv_heads = c.kv_heads; d.dim = c.dim; d.vdim = c.vdim; d.rot_pairs = c.rot_pairs; d.window = c.window;
    d.shared = shared(); d.scale = c.score_scale; d.softcap = c.softcap; d.eps = eps; d.proj = proj; d.ld = ld; d.k_off = q_cols(); d.v_off = q_cols() + k_cols();
    d.q_norm = f32(w[kWAux0]); d.k_norm = shared() ? nullptr : f32(w[kWAux1]); d.rot_table = reinterpret_cast<const float2*>(w[kWAux2].data());
    d.seq_stride = (int64_t)max_len * cld();
    d.cache = static_cast<uint8_t*>(mem) + (size_t)x.slot0 * cache_bytes(max_len);
    d.pos = pos; d.max_len = max_len; d.y = y; d.y_ld = y_ld;
    {
      Span span("grouped_append", esz * (double)x.rows() * 2.0 * (c.heads * c.dim + (shared() ? 0 : c.kv_heads * (c.dim + c.vdim))));
      AG_RETURN_IF_ERROR(k::grouped_append(x.s, d));
    }
    *launches += 1;
    if (x.T <= kShortT) {
      double keys = 0;
      for (int i = 0; i < x.n_seq; i++) keys += c.window ? std::min(c.window + x.T - 1, x.host_len[i] + x.T) : x.host_len[i] + x.T;
      Span span("grouped_decode", esz * (keys * c.kv_heads + (double)x.rows() * c.heads) * (c.dim + c.vdim));
      *launches += 1;
      return k::grouped_decode(x.s, d);
    }
    // sequences that hold equally many tokens share a launch
    for (int i = 0; i < x.n_seq;) {
      int n = 1;
      while (i + n < x.n_seq && x.host_len[i + n] == x.host_len[i]) n++;
      const uint8_t* cache = static_cast<const uint8_t*>(d.cache) + (size_t)i * cache_bytes(max_len);
      k::PromptAttnDesc p;
      p.dtype = dtype; p.n_seq = n; p.T = x.T; p.past = x.host_len[i]; p.heads = c.heads; p.group = c.heads / c.kv_heads; p.dim = c.dim; p.vdim = c.vdim; p.window = c.window;
      p.scale = c.score_scale; p.softcap = c.softcap;
      p.q = static_cast<const uint8_t*>(proj) + (size_t)i * x.T * ld * esz; p.q_ld = ld; p.q_b = x.T * ld;
      p.k = cache; p.v = cache + (size_t)k::grouped_v_col(c.kv_heads, c.dim) * esz; p.k_ld = p.v_ld = cld(); p.k_b = p.v_b = d.seq_stride;
      p.y = static_cast<uint8_t*>(y) + (size_t)i * x.T * y_ld * esz; p.y_ld = y_ld; p.y_b = x.T * y_ld;
      Span span("grouped_prefill", 2.0 * n * c.heads * (c.dim + c.vdim) * pairs_seen(p.past, x.T));
      AG_RETURN_IF_ERROR(k::prompt_attention(x.s, p));
      *launches += 1;
      i += n;
    }
    return Status::OK();
  }
};

struct LayerRun { int layer; int pass; bool first; int memory; };   // pass -1 outside the loop; memory: the run whose memory it uses

struct SeqEngine {
  SeqModelCfg cfg;
  DType dtype = DType::F32;
  std::vector<TensorRec> w;
  std::vector<std::unique_ptr<Mixer>> mixers;
  std::vector<LayerRun> runs;
  std::vector<std::shared_ptr<Buffer>> memory;     // per layer run, all slots (none where a run uses another one's)
  int slots = 0, max_len = 0;
  std::vector<int> len;                            // host mirror of pos
  Scratch pos, tok, history, step, rowmap, x, h1, h2, proj, gates, gu, cat, sub, work, kv, logits, picked;
  std::map<std::pair<int, int>, cudaGraphExec_t> graphs;
  int launches = 0, step_launches = 0;
  bool last_graph = false;

  ~SeqEngine() { drop_graphs(); }
  void drop_graphs() { for (auto& g : graphs) if (g.second) cudaGraphExecDestroy(g.second); graphs.clear(); }

  size_t esz() const { return dtype_size(dtype); }
  const TensorRec* lw(int l) const { return &w[4 + (size_t)l * kSeqLayerWeights]; }
  int64_t y_cols(const SeqLayerCfg& c) const { return pad8((int64_t)c.heads * c.vdim); }       // where the feed-forward's columns start
  bool sequential() const { return cfg.form == LayerForm::Sequential; }
  int64_t cat_k(const SeqLayerCfg& c) const { return c.ff && !sequential() ? y_cols(c) + c.ff : (int64_t)c.heads * c.vdim; }
  int64_t cat_ld(const SeqLayerCfg& c) const { return pad8(cat_k(c)); }

  // Grows a buffer (by half at least); graphs hold the old addresses of the buffers their step uses, so they are dropped and
  // recorded again.
  Status ensure(Scratch* b, size_t bytes, bool zero = false, bool in_graphs = true) {
    if (b->buf && b->buf->capacity >= bytes) return Status::OK();
    cudaStream_t s = DeviceCtx::get().stream;
    if (b->buf) {
      bytes = std::max(bytes, b->buf->capacity + b->buf->capacity / 2);
      if (in_graphs) { cudaStreamSynchronize(s); drop_graphs(); }
    }
    b->buf.reset();
    AG_RETURN_IF_ERROR(Shared::get().pool.acquire(bytes, &b->buf));
    if (zero && cudaMemsetAsync(b->buf->ptr, 0, b->buf->capacity, s) != cudaSuccess) return Status::compute("sequence engine: clear");
    return Status::OK();
  }
  Status reserve(int slot0, int n_seq, int T, int n_want) {
    const size_t R = (size_t)n_seq * T;
    int64_t pc = 0, gc = 1, fc = 1, cc = 0; size_t wb = 256, kb = 256;
    for (size_t l = 0; l < cfg.layers.size(); l++) {
      const SeqLayerCfg& c = cfg.layers[l];
      pc = std::max(pc, pad8(mixers[l]->proj_cols())); gc = std::max<int64_t>(gc, mixers[l]->gate_cols());
      fc = std::max(fc, k::glu_rows(c.ff)); cc = std::max({cc, cat_ld(c), pad8(c.ff)});
      wb = std::max(wb, mixers[l]->work_bytes(n_seq, T, max_len));
      if (T > kShortT) kb = std::max(kb, mixers[l]->kv_bytes(len.data() + slot0, n_seq, T));
    }
    AG_RETURN_IF_ERROR(ensure(&x, R * cfg.width * sizeof(float)));
    AG_RETURN_IF_ERROR(ensure(&proj, R * pc * esz()));
    AG_RETURN_IF_ERROR(ensure(&gates, R * gc * sizeof(float)));
    AG_RETURN_IF_ERROR(ensure(&cat, R * cc * esz(), true));
    if (sequential()) AG_RETURN_IF_ERROR(ensure(&sub, R * cfg.width * sizeof(float)));
    AG_RETURN_IF_ERROR(ensure(&work, wb));
    AG_RETURN_IF_ERROR(ensure(&kv, kb, false, false));
    const size_t hrows = std::max<size_t>(R, (size_t)n_want);
    AG_RETURN_IF_ERROR(ensure(&h1, hrows * pad8(cfg.width) * esz(), true));
    AG_RETURN_IF_ERROR(ensure(&h2, hrows * pad8(cfg.width) * esz(), true));
    if (R > k::kSeqSkinnyRows || !skinny_ok()) AG_RETURN_IF_ERROR(ensure(&gu, R * fc * esz()));
    if (n_want) AG_RETURN_IF_ERROR(ensure(&logits, (size_t)n_want * cfg.vocab * sizeof(float)));
    AG_RETURN_IF_ERROR(ensure(&tok, std::max<size_t>(R, slots) * sizeof(int32_t)));
    AG_RETURN_IF_ERROR(ensure(&rowmap, std::max<size_t>(R, 64) * sizeof(int32_t)));
    return Status::OK();
  }
  bool skinny_ok() const {
    int64_t kmax = cfg.width;
    for (const SeqLayerCfg& c : cfg.layers) kmax = std::max({kmax, cat_k(c), (int64_t)c.ff});
    return k::seq_skinny_fits(kmax);
  }

  Status count(Status st) { launches++; return st; }

  void* mem_of(const LayerRun& run) const { return memory[run.memory]->ptr; }
  // One product of a sequential layer: rows of `a` against wt, by the kernel the number of rows calls for.
  Status enqueue_product(const StepCtx& st, const char* name, const void* a, int64_t a_ld, int64_t kdim, const TensorRec& wt, int64_t n, void* out, int64_t out_ld, bool out_f32,
                         bool bytes = false) {
    const int R = st.rows();
    Span span(name, R <= k::kSeqSkinnyRows ? esz() * (double)n * pad8(kdim) : bytes ? R * (esz() * kdim + 4.0 * n) : product(R, n, kdim));
    if (R <= k::kSeqSkinnyRows && skinny_ok()) {
      k::SeqSkinnyDesc d;
      d.dtype = dtype; d.rows = R; d.k = (int)kdim; d.a = a; d.a_ld = a_ld; d.n_seg = 1;
      k::SeqSeg& g = d.seg[0];
      g.a = a; g.a_ld = a_ld; g.w = wt.data(); g.ld = pad8(kdim); g.n = (int)n; g.mode = out_f32 ? k::SeqOut::StoreF32 : k::SeqOut::Store; g.out = out; g.out_ld = out_ld;
      return count(k::seq_skinny(st.s, d));
    }
    return count(k::matmul(st.s, linear_desc(dtype, a, a_ld, R, kdim, wt.data(), pad8(kdim), n, out, out_ld, out_f32, nullptr)));
  }
  // The gated half of a feed-forward: out [R, ff] from the normed rows in h.
  Status enqueue_glu(const StepCtx& st, const SeqLayerCfg& c, const void* h, const TensorRec& wt, void* out, int64_t out_ld) {
    const int R = st.rows();
    const int64_t wl = pad8(cfg.width), fn = k::glu_rows(c.ff);
    if (R <= k::kSeqSkinnyRows && skinny_ok()) {
      k::SeqSkinnyDesc d;
      d.dtype = dtype; d.rows = R; d.k = cfg.width; d.a = h; d.a_ld = wl; d.n_seg = 1;
      k::SeqSeg& g = d.seg[0];
      g.a = h; g.a_ld = wl; g.w = wt.data(); g.ld = wl; g.n = c.ff; g.mode = k::SeqOut::Glu; g.glu = (k::Glu)c.glu; g.limit = c.ff_limit; g.out = out; g.out_ld = out_ld;
      Span span("skinny_ff", esz() * 2.0 * c.ff * wl);
      return count(k::seq_skinny(st.s, d));
    }
    k::GemmDesc g = linear_desc(dtype, h, wl, R, cfg.width, wt.data(), wl, fn, gu.ptr(), fn, false, nullptr);
    Span span("linear_ff", product(R, 2.0 * c.ff, cfg.width));
    if (k::matmul_tc_ready(g)) {                          // the gate rides in the product's epilogue
      g.c = out; g.c_row = out_ld; g.ep.glu_n = c.ff; g.ep.glu = (k::Glu)c.glu; g.ep.glu_limit = c.ff_limit;
      return count(k::matmul(st.s, g));
    }
    AG_RETURN_IF_ERROR(count(k::matmul(st.s, g)));
    return count(k::glu(st.s, dtype, gu.ptr(), fn, out, out_ld, R, c.ff, k::kGluBlock, (k::Glu)c.glu, c.ff_limit));
  }
  // A sequential layer leaves its last sublayer's output in `sub`; *post is the weight of the norm through which the next norm
  // kernel adds it to the stream.
  Status enqueue_sequential(const StepCtx& st, const LayerRun& run, bool start, const float** post) {
    const int R = st.rows();
    float* X = static_cast<float*>(x.ptr());
    const SeqLayerCfg& c = cfg.layers[run.layer];
    const Mixer& mx = *mixers[run.layer];
    const TensorRec* W = lw(run.layer);
    const int64_t pl = pad8(mx.proj_cols()), cl = cat_ld(c), wl = pad8(cfg.width);
    auto norm = [&](const TensorRec& w1, bool first) {
      k::RmsRowsDesc n;
      n.dtype = dtype; n.x = X; n.rows = R; n.width = cfg.width; n.eps = cfg.eps; n.w1 = f32(w1); n.out1 = h1.ptr(); n.ld1 = wl;
      if (first && (start || (run.first && run.pass > 0))) {
        n.tok = static_cast<const int32_t*>(tok.ptr()); n.embed = w[0].data(); n.embed_ld = w[0].shape[1]; n.vocab = cfg.vocab; n.embed_scale = cfg.embed_scale;
        n.load_x = !start;
      }
      if (first && run.first) n.step = f32(w[3]) + (size_t)run.pass * cfg.width;
      if (*post) { n.post = static_cast<const float*>(sub.ptr()); n.post_w = *post; }
      *post = nullptr;
      Span span("rms_rows", (double)R * cfg.width * ((n.post ? 12.0 : 4.0) + esz()));
      return count(k::rms_rows(st.s, n));
    };
    AG_RETURN_IF_ERROR(norm(W[kWNorm1], true));
    if (mx.gate_cols() && R <= k::kSeqSkinnyRows && skinny_ok()) {          // both input products in one launch
      k::SeqSkinnyDesc d;
      d.dtype = dtype; d.rows = R; d.k = cfg.width; d.a = h1.ptr(); d.a_ld = wl; d.n_seg = 2;
      for (int i = 0; i < 2; i++) { d.seg[i].a = h1.ptr(); d.seg[i].a_ld = wl; d.seg[i].ld = wl; }
      d.seg[0].w = W[kWIn].data(); d.seg[0].n = mx.proj_cols(); d.seg[0].mode = k::SeqOut::Store; d.seg[0].out = proj.ptr(); d.seg[0].out_ld = pl;
      d.seg[1].w = W[kWAux0].data(); d.seg[1].n = mx.gate_cols(); d.seg[1].mode = k::SeqOut::StoreF32; d.seg[1].out = gates.ptr(); d.seg[1].out_ld = mx.gate_cols();
      Span span("skinny_in", esz() * (double)wl * (mx.proj_cols() + mx.gate_cols()));
      AG_RETURN_IF_ERROR(count(k::seq_skinny(st.s, d)));
    } else {
      AG_RETURN_IF_ERROR(enqueue_product(st, R <= k::kSeqSkinnyRows ? "skinny_in" : "linear_in", h1.ptr(), wl, cfg.width, W[kWIn], mx.proj_cols(), proj.ptr(), pl, false));
      if (mx.gate_cols()) AG_RETURN_IF_ERROR(enqueue_product(st, "linear_gates", h1.ptr(), wl, cfg.width, W[kWAux0], mx.gate_cols(), gates.ptr(), mx.gate_cols(), true, true));
    }
    AG_RETURN_IF_ERROR(mx.run(st, proj.ptr(), pl, static_cast<const float*>(gates.ptr()), mem_of(run), max_len, static_cast<const int*>(pos.ptr()) + st.slot0, cat.ptr(), cl, work.ptr(),
                              kv.ptr(), cfg.eps, &launches));
    AG_RETURN_IF_ERROR(enqueue_product(st, R <= k::kSeqSkinnyRows ? "skinny_out" : "linear_out", cat.ptr(), cl, cat_k(c), W[kWOut], cfg.width, sub.ptr(), cfg.width, true));
    *post = f32(W[kWPost1]);
    if (!c.ff) return Status::OK();
    AG_RETURN_IF_ERROR(norm(W[kWNorm2], false));
    AG_RETURN_IF_ERROR(enqueue_glu(st, c, h1.ptr(), W[kWFf], cat.ptr(), pad8(c.ff)));
    AG_RETURN_IF_ERROR(enqueue_product(st, R <= k::kSeqSkinnyRows ? "skinny_out" : "linear_out", cat.ptr(), pad8(c.ff), c.ff, W[kWDown], cfg.width, sub.ptr(), cfg.width, true));
    *post = f32(W[kWPost2]);
    return Status::OK();
  }
  Status enqueue_parallel(const StepCtx& st, const LayerRun& run, bool start) {
    const int R = st.rows();
    const bool skinny = R <= k::kSeqSkinnyRows && skinny_ok();
    float* X = static_cast<float*>(x.ptr());
    const int* p = static_cast<const int*>(pos.ptr()) + st.slot0;
    const SeqLayerCfg& c = cfg.layers[run.layer];
    const Mixer& mx = *mixers[run.layer];
    const TensorRec* W = lw(run.layer);
    const int64_t pl = pad8(mx.proj_cols()), cl = cat_ld(c), wl = pad8(cfg.width);
    uint8_t* ff_out = static_cast<uint8_t*>(cat.ptr()) + (size_t)y_cols(c) * esz();
    // what happens to the stream ahead of this run rides in the norm: the embedding, a pass's additions
    k::RmsRowsDesc n;
    n.dtype = dtype; n.x = X; n.rows = R; n.width = cfg.width; n.eps = cfg.eps;
    const bool again = run.first && run.pass > 0;
    if (start || again) { n.tok = static_cast<const int32_t*>(tok.ptr()); n.embed = w[0].data(); n.embed_ld = w[0].shape[1]; n.vocab = cfg.vocab; n.embed_scale = cfg.embed_scale; }
    n.load_x = !start;
    if (run.first) n.step = f32(w[3]) + (size_t)run.pass * cfg.width;
    if (skinny) {
      // 16-bit: the norms are stored once and every product reads them; float32: the products take them in their prologue
      const bool stored = dtype != DType::F32;
      if (stored) {
        n.w1 = f32(W[kWNorm1]); n.out1 = h1.ptr(); n.ld1 = wl;
        if (c.ff) { n.w2 = f32(W[kWNorm2]); n.out2 = h2.ptr(); n.ld2 = wl; }
      }
      if (stored || start || n.step) AG_RETURN_IF_ERROR(count(k::rms_rows(st.s, n)));
      k::SeqSkinnyDesc d;
      d.dtype = dtype; d.rows = R; d.k = cfg.width; d.eps = cfg.eps;
      if (!stored) d.x = X;
      auto seg = [&](const TensorRec& wt, int64_t cols, const TensorRec& nw, const Scratch& h, k::SeqOut mode, void* out, int64_t ld) {
        k::SeqSeg& g = d.seg[d.n_seg++];
        g.w = wt.data(); g.ld = wl; g.n = (int)cols; g.mode = mode; g.glu = (k::Glu)c.glu; g.limit = c.ff_limit; g.out = out; g.out_ld = ld;
        if (stored) { g.a = h.ptr(); g.a_ld = wl; } else g.norm_w = f32(nw);
      };
      seg(W[kWIn], mx.proj_cols(), W[kWNorm1], h1, k::SeqOut::Store, proj.ptr(), pl);
      if (mx.gate_cols()) seg(W[kWAux0], mx.gate_cols(), W[kWNorm1], h1, k::SeqOut::StoreF32, gates.ptr(), mx.gate_cols());
      if (c.ff) seg(W[kWFf], c.ff, W[kWNorm2], h2, k::SeqOut::Glu, ff_out, cl);
      Span span("skinny_in", esz() * (double)wl * (mx.proj_cols() + mx.gate_cols() + 2.0 * c.ff));
      AG_RETURN_IF_ERROR(count(k::seq_skinny(st.s, d)));
    } else {
      n.w1 = f32(W[kWNorm1]); n.out1 = h1.ptr(); n.ld1 = wl;
      if (c.ff) { n.w2 = f32(W[kWNorm2]); n.out2 = h2.ptr(); n.ld2 = wl; }
      {
        Span span("rms_rows", (4.0 + (c.ff ? 2.0 : 1.0) * esz()) * R * cfg.width);
        AG_RETURN_IF_ERROR(count(k::rms_rows(st.s, n)));
      }
      {
        Span span("linear_in", product(R, mx.proj_cols(), cfg.width));
        AG_RETURN_IF_ERROR(count(k::matmul(st.s, linear_desc(dtype, h1.ptr(), wl, R, cfg.width, W[kWIn].data(), wl, mx.proj_cols(), proj.ptr(), pl, false, nullptr))));
      }
      if (mx.gate_cols()) {
        Span span("linear_gates", (double)R * (esz() * cfg.width + 4.0 * mx.gate_cols()));      // bound by reading its input
        AG_RETURN_IF_ERROR(count(k::matmul(st.s, linear_desc(dtype, h1.ptr(), wl, R, cfg.width, W[kWAux0].data(), wl, mx.gate_cols(), gates.ptr(), mx.gate_cols(), true, nullptr))));
      }
      if (c.ff) {
        const int64_t fn = k::glu_rows(c.ff);
        k::GemmDesc g = linear_desc(dtype, h2.ptr(), wl, R, cfg.width, W[kWFf].data(), wl, fn, gu.ptr(), fn, false, nullptr);
        if (k::matmul_tc_ready(g)) {                  // the gate rides in the product's epilogue
          g.c = ff_out; g.c_row = cl; g.ep.glu_n = c.ff; g.ep.glu = (k::Glu)c.glu; g.ep.glu_limit = c.ff_limit;
          Span span("linear_ff", product(R, 2.0 * c.ff, cfg.width));
          AG_RETURN_IF_ERROR(count(k::matmul(st.s, g)));
        } else {
          {
            Span span("linear_ff", product(R, 2.0 * c.ff, cfg.width));
            AG_RETURN_IF_ERROR(count(k::matmul(st.s, g)));
          }
          Span span("clamped_glu", 3.0 * esz() * R * c.ff);
          AG_RETURN_IF_ERROR(count(k::glu(st.s, dtype, gu.ptr(), fn, ff_out, cl, R, c.ff, k::kGluBlock, (k::Glu)c.glu, c.ff_limit)));
        }
      }
    }
    AG_RETURN_IF_ERROR(mx.run(st, proj.ptr(), pl, static_cast<const float*>(gates.ptr()), mem_of(run), max_len, p, cat.ptr(), cl, work.ptr(), kv.ptr(), cfg.eps, &launches));
    if (skinny) {
      k::SeqSkinnyDesc d;
      d.dtype = dtype; d.rows = R; d.k = (int)cat_k(c); d.a = cat.ptr(); d.a_ld = cl; d.n_seg = 1;
      d.seg[0].a = cat.ptr(); d.seg[0].a_ld = cl;
      d.seg[0].w = W[kWOut].data(); d.seg[0].ld = cl; d.seg[0].n = cfg.width; d.seg[0].mode = k::SeqOut::AddF32; d.seg[0].out = X; d.seg[0].out_ld = cfg.width;
      Span span("skinny_out", esz() * (double)cl * cfg.width);
      AG_RETURN_IF_ERROR(count(k::seq_skinny(st.s, d)));
    } else {
      Span span("linear_out", product(R, cfg.width, cat_k(c)));
      AG_RETURN_IF_ERROR(count(k::matmul(st.s, linear_desc(dtype, cat.ptr(), cl, R, cat_k(c), W[kWOut].data(), cl, cfg.width, X, cfg.width, true, X))));
    }
    return Status::OK();
  }

  // All layers over the R rows whose tokens are in `tok`; x holds the residual stream afterwards, but for what *post (see
  // enqueue_sequential) says is still to be added.
  Status enqueue_layers(const StepCtx& st, float* layers_out, const float** post) {
    const size_t R = (size_t)st.rows();
    *post = nullptr;
    for (size_t r = 0; r < runs.size(); r++) {
      AG_RETURN_IF_ERROR(sequential() ? enqueue_sequential(st, runs[r], r == 0, post) : enqueue_parallel(st, runs[r], r == 0));
      if (layers_out) {
        if (*post) {
          k::RmsRowsDesc n;
          n.dtype = dtype; n.x = static_cast<float*>(x.ptr()); n.rows = R; n.width = cfg.width; n.eps = cfg.eps; n.post = static_cast<const float*>(sub.ptr()); n.post_w = *post;
          *post = nullptr;
          AG_RETURN_IF_ERROR(count(k::rms_rows(st.s, n)));
        }
        cudaError_t e = cudaMemcpyAsync(layers_out + r * R * cfg.width, x.ptr(), R * cfg.width * sizeof(float), cudaMemcpyDeviceToHost, st.s);
        if (e != cudaSuccess) return Status::compute("sequence engine: layer copy");
      }
    }
    return Status::OK();
  }

  // Logits of n rows of x: all of them in order (map null), or the ones listed in the device array `map`; post: as enqueue_layers left it.
  Status enqueue_head(cudaStream_t s, int n, const int32_t* map, const float* post) {
    const int64_t wl = pad8(cfg.width);
    Span span(n <= k::kSeqSkinnyRows ? "skinny_head" : "linear_head", n <= k::kSeqSkinnyRows ? esz() * (double)wl * cfg.vocab : product(n, cfg.vocab, cfg.width));
    const bool skinny = n <= k::kSeqSkinnyRows && k::seq_skinny_fits(cfg.width);
    k::SeqSkinnyDesc d;
    d.dtype = dtype; d.rows = n; d.k = cfg.width; d.eps = cfg.eps; d.n_seg = 1;
    d.seg[0].w = w[1].data(); d.seg[0].ld = wl; d.seg[0].n = cfg.vocab; d.seg[0].norm_w = f32(w[2]); d.seg[0].mode = k::SeqOut::StoreF32; d.seg[0].out = logits.ptr();
    d.seg[0].out_ld = cfg.vocab;
    if (skinny && !map && !post && dtype == DType::F32) { d.x = static_cast<const float*>(x.ptr()); return count(k::seq_skinny(s, d)); }
    k::RmsRowsDesc r;
    r.dtype = dtype; r.x = static_cast<float*>(x.ptr()); r.rows = n; r.width = cfg.width; r.eps = cfg.eps; r.row_map = map; r.w1 = f32(w[2]); r.out1 = h1.ptr(); r.ld1 = wl;
    if (post) { r.post = static_cast<const float*>(sub.ptr()); r.post_w = post; }
    AG_RETURN_IF_ERROR(count(k::rms_rows(s, r)));
    if (skinny) { d.a = d.seg[0].a = h1.ptr(); d.a_ld = d.seg[0].a_ld = wl; return count(k::seq_skinny(s, d)); }
    return count(k::matmul(s, linear_desc(dtype, h1.ptr(), wl, n, cfg.width, w[1].data(), wl, cfg.vocab, logits.ptr(), cfg.vocab, true, nullptr)));
  }
  Status enqueue_pick(cudaStream_t s, int n, void* out) {
    return count(k::argmax(s, TView::make(logits.ptr(), DType::F32, {(int64_t)n, (int64_t)cfg.vocab}), TView::make(out, DType::I32, {(int64_t)n})));
  }

  // One token per sequence: consumes tok[0 .. n), leaves the logits, the greedy choice in tok and in the history.
  Status enqueue_step(cudaStream_t s, int slot0, int n) {
    launches = 0;
    StepCtx st{s, slot0, n, 1, len.data() + slot0};
    const float* post = nullptr;
    AG_RETURN_IF_ERROR(enqueue_layers(st, nullptr, &post));
    AG_RETURN_IF_ERROR(enqueue_head(s, n, nullptr, post));
    AG_RETURN_IF_ERROR(enqueue_pick(s, n, tok.ptr()));
    AG_RETURN_IF_ERROR(count(k::seq_advance(s, static_cast<int*>(pos.ptr()) + slot0, n, 1, static_cast<const int32_t*>(tok.ptr()), static_cast<int32_t*>(history.ptr()),
                                            static_cast<int*>(step.ptr()), max_len)));
    step_launches = launches;
    return Status::OK();
  }
  // Runs one such step: the first one of a slot range launch by launch (one-time kernel attributes are set outside any
  // capture), the second one is captured, later ones replay the graph.
  Status run_step(cudaStream_t s, int slot0, int n, bool use_graph) {
    last_graph = false;
    if (!use_graph || profile::enabled()) { AG_RETURN_IF_ERROR(enqueue_step(s, slot0, n)); }
    else {
      const auto key = std::make_pair(slot0, n);
      auto it = graphs.find(key);
      if (it == graphs.end()) { graphs[key] = nullptr; AG_RETURN_IF_ERROR(enqueue_step(s, slot0, n)); }
      else {
        if (!it->second) {
          cudaGraph_t g = nullptr;
          Status st = Status::OK();
          if (cudaStreamBeginCapture(s, cudaStreamCaptureModeRelaxed) == cudaSuccess) {
            st = enqueue_step(s, slot0, n);
            const cudaError_t ce = cudaStreamEndCapture(s, &g);
            if (!(st.ok() && ce == cudaSuccess && g && cudaGraphInstantiate(&it->second, g, 0) == cudaSuccess)) { it->second = nullptr; cudaGetLastError(); }
            if (g) cudaGraphDestroy(g);
          } else cudaGetLastError();
          if (!st.ok()) return st;
        }
        if (it->second) {
          const cudaError_t e = cudaGraphLaunch(it->second, s);
          if (e != cudaSuccess) return Status::compute(std::string("sequence engine: graph launch: ") + cudaGetErrorString(e));
          last_graph = true;
        } else AG_RETURN_IF_ERROR(enqueue_step(s, slot0, n));
      }
    }
    g_launch_count.fetch_add((uint64_t)step_launches, std::memory_order_relaxed);
    for (int i = 0; i < n; i++) len[slot0 + i]++;
    return Status::OK();
  }
};

std::mutex g_seq_mu;
std::unordered_map<uint64_t, std::unique_ptr<SeqEngine>> g_seq;
uint64_t g_seq_next = 1;
SeqEngine* find(uint64_t h) { auto it = g_seq.find(h); return it == g_seq.end() ? nullptr : it->second.get(); }

Status finish(cudaStream_t s) {
  k::status_snapshot(s, 0);
  const cudaError_t e = cudaStreamSynchronize(s);
  if (e != cudaSuccess) return Status::compute(std::string("synchronize: ") + cudaGetErrorString(e));
  const int code = k::status_take(s, 0);
  if (code != 0) return Status::compute("tensor-core pipeline wait timed out (code " + std::to_string(code) + ")");
  return Status::OK();
}

Status check_slots(const SeqEngine* e, int slot0, int n) {
  if (slot0 < 0 || n < 1 || slot0 + n > e->slots) return Status::invalid("sequence engine: no such slot");
  return Status::OK();
}

}  // namespace

Status seq_create(const SeqModelCfg& cfg, const std::vector<TensorRec>& weights, int slots, int max_len, uint64_t* handle) {
  DeviceCtx& ctx = DeviceCtx::get();
  if (ctx.dry) return Status::compute("no CUDA device (dry-run mode)");
  const int n_layers = (int)cfg.layers.size();
  if (cfg.vocab < 1 || cfg.width < 1 || n_layers < 1 || slots < 1 || max_len < 1) return Status::invalid("sequence model: bad configuration");
  if (cfg.loop_times < 0 || (cfg.loop_times && (cfg.loop_start < 0 || cfg.loop_stop <= cfg.loop_start || cfg.loop_stop > n_layers)))
    return Status::invalid("sequence model: bad loop");
  if (weights.size() != 4 + (size_t)n_layers * kSeqLayerWeights) return Status::invalid("sequence model: wrong number of weights");
  auto e = std::make_unique<SeqEngine>();
  e->cfg = cfg; e->w = weights; e->slots = slots; e->max_len = max_len; e->dtype = weights[0].dtype;
  const DType dt = e->dtype;
  if (!(dt == DType::F32 || dt == DType::F16 || dt == DType::BF16)) return Status::unsupported("sequence model: float weights only");
  const int64_t W = cfg.width, wl = pad8(W);
  if (!is_matrix(weights[0], dt, cfg.vocab, W) || !is_matrix(weights[1], dt, cfg.vocab, wl) || !is_vector(weights[2], W)) return Status::invalid("sequence model: embedding, head or final norm");
  if (cfg.loop_times && !is_vector(weights[3], (int64_t)cfg.loop_times * W)) return Status::invalid("sequence model: step vectors");
  for (int l = 0; l < n_layers; l++) {
    const SeqLayerCfg& c = e->cfg.layers[l];
    const TensorRec* t = e->lw(l);
    const std::string at = "sequence model: layer " + std::to_string(l) + ": ";
    if (c.heads < 1 || c.dim < 1 || c.vdim < 1 || c.ff < 0) return Status::invalid(at + "bad sizes");
    if (c.mixer == MixerKind::Mlstm) e->mixers.emplace_back(new MlstmMixer(c, t, dt));
    else if (c.mixer == MixerKind::LatentAttention) e->mixers.emplace_back(new LatentMixer(c, t, dt));
    else if (c.mixer == MixerKind::KeyDecay) e->mixers.emplace_back(new KeyDecayMixer(c, t, dt));
    else if (c.mixer == MixerKind::GroupedAttention) e->mixers.emplace_back(new GroupedMixer(c, t, dt));
    else return Status::invalid(at + "unknown mixer");
    const Mixer& m = *e->mixers.back();
    if (!is_vector(t[kWNorm1], W) || !is_matrix(t[kWIn], dt, m.proj_cols(), wl) || !is_matrix(t[kWOut], dt, W, e->cat_ld(c))) return Status::invalid(at + "norm, input or output weights");
    if (c.ff && (!is_vector(t[kWNorm2], W) || !is_matrix(t[kWFf], dt, k::glu_rows(c.ff), wl))) return Status::invalid(at + "feed-forward weights");
    if (e->sequential() && (!is_vector(t[kWPost1], W) || (c.ff && (!is_vector(t[kWPost2], W) || !is_matrix(t[kWDown], dt, W, pad8(c.ff))))))
      return Status::invalid(at + "norms behind the sublayers or feed-forward output");
    if (c.kv_from >= l) return Status::invalid(at + "keys come from an earlier layer");
    const Status st = m.check(cfg, max_len);
    if (!st.ok()) return Status{st.kind, at + st.msg};
  }
  auto add = [&](int lo, int hi, int pass) { for (int l = lo; l < hi; l++) e->runs.push_back({l, pass, pass >= 0 && l == lo, (int)e->runs.size()}); };
  if (cfg.loop_times) {
    add(0, cfg.loop_start, -1);
    for (int t = 0; t < cfg.loop_times; t++) add(cfg.loop_start, cfg.loop_stop, t);
    add(cfg.loop_stop, n_layers, -1);
  } else add(0, n_layers, -1);
  for (size_t i = 0; i < e->runs.size(); i++) {         // keys of another layer: its latest run
    const int from = e->cfg.layers[e->runs[i].layer].kv_from;
    if (from < 0) continue;
    size_t j = i;
    while (j > 0 && e->runs[j].layer != from) j--;
    if (e->runs[j].layer != from) return Status::invalid("sequence model: keys come from a layer that has not run");
    e->runs[i].memory = (int)j;
  }
  for (const LayerRun& r : e->runs) {
    std::shared_ptr<Buffer> b;
    if (e->mixers[r.layer]->slot_bytes(max_len) == 0) { e->memory.push_back(nullptr); continue; }
    AG_RETURN_IF_ERROR(Shared::get().pool.acquire((size_t)slots * e->mixers[r.layer]->slot_bytes(max_len), &b));
    // padding columns of caches take part in products with zeros: they must hold numbers
    if (cudaMemsetAsync(b->ptr, 0, b->capacity, ctx.stream) != cudaSuccess) return Status::compute("sequence engine: clear");
    e->memory.push_back(b);
  }
  e->len.assign(slots, 0);
  AG_RETURN_IF_ERROR(e->ensure(&e->pos, (size_t)slots * sizeof(int), true));
  AG_RETURN_IF_ERROR(e->ensure(&e->step, 256, true));
  AG_RETURN_IF_ERROR(e->ensure(&e->history, (size_t)max_len * slots * sizeof(int32_t)));
  AG_RETURN_IF_ERROR(e->ensure(&e->picked, (size_t)kMaxRows * sizeof(int32_t)));
  std::lock_guard<std::mutex> g(g_seq_mu);
  *handle = g_seq_next++;
  g_seq[*handle] = std::move(e);
  return seq_reset(*handle, 0, -1);
}

// Gives slots back empty: recurrent states start at zero, cached rows beyond the length are never read. n < 0: all slots
// (called with the lock held by seq_create).
Status seq_reset(uint64_t handle, int slot, int n) {
  std::unique_lock<std::mutex> g(g_seq_mu, std::defer_lock);
  if (n >= 0) g.lock();
  SeqEngine* e = find(handle);
  if (!e) return Status::invalid("sequence engine: unknown handle");
  if (n < 0) { slot = 0; n = e->slots; }
  AG_RETURN_IF_ERROR(check_slots(e, slot, n));
  cudaStream_t s = DeviceCtx::get().stream;
  cudaError_t err = cudaMemsetAsync(static_cast<int*>(e->pos.ptr()) + slot, 0, (size_t)n * sizeof(int), s);
  for (size_t r = 0; r < e->runs.size() && err == cudaSuccess; r++) {
    const Mixer& m = *e->mixers[e->runs[r].layer];
    if (!m.clear_on_reset()) continue;
    const size_t b = m.slot_bytes(e->max_len);
    err = cudaMemsetAsync(static_cast<uint8_t*>(e->memory[r]->ptr) + (size_t)slot * b, 0, (size_t)n * b, s);
  }
  if (err != cudaSuccess) return Status::compute(std::string("sequence engine: reset: ") + cudaGetErrorString(err));
  for (int i = 0; i < n; i++) e->len[slot + i] = 0;
  return Status::OK();
}

Status seq_forward(uint64_t handle, int slot0, int n_seq, const int32_t* tokens, int T, const int32_t* want, int n_want, float* host_logits, int32_t* picked,
                   float* layers_out) {
  std::lock_guard<std::mutex> g(g_seq_mu);
  SeqEngine* e = find(handle);
  if (!e) return Status::invalid("sequence engine: unknown handle");
  AG_RETURN_IF_ERROR(check_slots(e, slot0, n_seq));
  if (T < 1 || !tokens || n_want < 0 || (n_want && !want)) return Status::invalid("sequence engine: bad step");
  for (int i = 0; i < n_seq; i++)
    if (e->len[slot0 + i] + T > e->max_len) return Status::limit("sequence engine: a sequence would outgrow its " + std::to_string(e->max_len) + " tokens");
  for (int64_t i = 0; i < (int64_t)n_seq * T; i++)
    if (tokens[i] < 0 || tokens[i] >= e->cfg.vocab) return Status::invalid("sequence engine: token id out of range");
  for (int i = 0; i < n_want; i++)
    if (want[i] < 0 || want[i] >= n_seq * T) return Status::invalid("sequence engine: wanted row out of range");
  DeviceCtx& ctx = DeviceCtx::get();
  AG_RETURN_IF_ERROR(ctx.make_current());
  cudaStream_t s = ctx.stream;
  const size_t V = (size_t)e->cfg.vocab;
  const int cut = std::max(1, kMaxRows / n_seq);
  if (layers_out && T > cut) return Status::invalid("sequence engine: the portion is too long to record its layers");
  auto copy_ok = [](cudaError_t c) { return c == cudaSuccess ? Status::OK() : Status::compute(std::string("sequence engine: copy: ") + cudaGetErrorString(c)); };
  for (int t0 = 0; t0 < T; t0 += cut) {
    const int t1 = std::min(T, t0 + cut), Ts = t1 - t0;
    std::vector<int32_t> toks((size_t)n_seq * Ts), rows, idx;
    for (int i = 0; i < n_seq; i++) std::copy(tokens + (size_t)i * T + t0, tokens + (size_t)i * T + t1, toks.begin() + (size_t)i * Ts);
    for (int i = 0; i < n_want; i++) {
      const int sq = want[i] / T, t = want[i] % T;
      if (t >= t0 && t < t1) { rows.push_back(sq * Ts + (t - t0)); idx.push_back(i); }
    }
    const int nw = (int)rows.size();
    bool in_order = nw == n_seq * Ts;
    for (int i = 0; i < nw && in_order; i++) in_order = rows[i] == i;
    const bool one_token = T == 1 && !layers_out && (nw == 0 || in_order);
    AG_RETURN_IF_ERROR(e->reserve(slot0, n_seq, Ts, one_token ? n_seq : nw));
    AG_RETURN_IF_ERROR(copy_ok(cudaMemcpyAsync(e->tok.ptr(), toks.data(), toks.size() * 4, cudaMemcpyHostToDevice, s)));
    if (one_token) {
      // the step greedy generation replays; the picked token is ignored unless asked for
      AG_RETURN_IF_ERROR(copy_ok(cudaMemsetAsync(e->step.ptr(), 0, sizeof(int), s)));
      AG_RETURN_IF_ERROR(e->run_step(s, slot0, n_seq, true));
      if (nw && picked) AG_RETURN_IF_ERROR(copy_ok(cudaMemcpyAsync(picked, e->tok.ptr(), (size_t)nw * 4, cudaMemcpyDeviceToHost, s)));
    } else {
      e->launches = 0;
      StepCtx st{s, slot0, n_seq, Ts, e->len.data() + slot0};
      const float* post = nullptr;
      AG_RETURN_IF_ERROR(e->enqueue_layers(st, layers_out, &post));
      if (nw) {
        if (!in_order) AG_RETURN_IF_ERROR(copy_ok(cudaMemcpyAsync(e->rowmap.ptr(), rows.data(), (size_t)nw * 4, cudaMemcpyHostToDevice, s)));
        AG_RETURN_IF_ERROR(e->enqueue_head(s, nw, in_order ? nullptr : static_cast<const int32_t*>(e->rowmap.ptr()), post));
        if (picked) {
          AG_RETURN_IF_ERROR(e->enqueue_pick(s, nw, e->picked.ptr()));
          std::vector<int32_t> got(nw);
          AG_RETURN_IF_ERROR(copy_ok(cudaMemcpyAsync(got.data(), e->picked.ptr(), (size_t)nw * 4, cudaMemcpyDeviceToHost, s)));
          AG_RETURN_IF_ERROR(copy_ok(cudaStreamSynchronize(s)));
          for (int i = 0; i < nw; i++) picked[idx[i]] = got[i];
        }
      }
      AG_RETURN_IF_ERROR(e->count(k::seq_advance(s, static_cast<int*>(e->pos.ptr()) + slot0, n_seq, Ts, nullptr, nullptr, nullptr, 0)));
      for (int i = 0; i < n_seq; i++) e->len[slot0 + i] += Ts;
      g_launch_count.fetch_add((uint64_t)e->launches, std::memory_order_relaxed);
    }
    if (host_logits) {
      for (int i = 0; i < nw;) {                       // runs of rows that lie together on both sides
        int j = i + 1;
        while (j < nw && idx[j] == idx[j - 1] + 1) j++;
        AG_RETURN_IF_ERROR(copy_ok(cudaMemcpyAsync(host_logits + (size_t)idx[i] * V, static_cast<float*>(e->logits.ptr()) + (size_t)i * V, (size_t)(j - i) * V * 4,
                                                   cudaMemcpyDeviceToHost, s)));
        i = j;
      }
    }
    AG_RETURN_IF_ERROR(finish(s));
  }
  if (picked && n_want == n_seq && T > 1) AG_RETURN_IF_ERROR(copy_ok(cudaMemcpy(e->tok.ptr(), picked, (size_t)n_seq * 4, cudaMemcpyHostToDevice)));
  return Status::OK();
}

Status seq_decode(uint64_t handle, int slot0, int n_seq, int n_steps, int32_t* host_tokens, bool use_graph) {
  std::lock_guard<std::mutex> g(g_seq_mu);
  SeqEngine* e = find(handle);
  if (!e) return Status::invalid("sequence engine: unknown handle");
  AG_RETURN_IF_ERROR(check_slots(e, slot0, n_seq));
  if (n_steps < 1 || !host_tokens) return Status::OK();
  for (int i = 0; i < n_seq; i++) {
    if (e->len[slot0 + i] < 1) return Status::invalid("sequence engine: no prompt yet");
    if (e->len[slot0 + i] + n_steps > e->max_len) return Status::limit("sequence engine: a sequence would outgrow its " + std::to_string(e->max_len) + " tokens");
  }
  DeviceCtx& ctx = DeviceCtx::get();
  AG_RETURN_IF_ERROR(ctx.make_current());
  cudaStream_t s = ctx.stream;
  AG_RETURN_IF_ERROR(e->reserve(slot0, n_seq, 1, n_seq));
  if (cudaMemsetAsync(e->step.ptr(), 0, sizeof(int), s) != cudaSuccess) return Status::compute("sequence engine: step counter");
  for (int i = 0; i < n_steps; i++) AG_RETURN_IF_ERROR(e->run_step(s, slot0, n_seq, use_graph));
  const cudaError_t ce = cudaMemcpyAsync(host_tokens, e->history.ptr(), (size_t)n_steps * n_seq * 4, cudaMemcpyDeviceToHost, s);
  if (ce != cudaSuccess) return Status::compute(std::string("sequence engine: tokens: ") + cudaGetErrorString(ce));
  return finish(s);
}

int seq_length(uint64_t handle, int slot) {
  std::lock_guard<std::mutex> g(g_seq_mu);
  SeqEngine* e = find(handle);
  return e && slot >= 0 && slot < e->slots ? e->len[slot] : -1;
}
int seq_info(uint64_t handle, int what) {
  std::lock_guard<std::mutex> g(g_seq_mu);
  SeqEngine* e = find(handle);
  if (!e) return -1;
  return what == 0 ? e->step_launches : what == 1 ? (e->last_graph ? 1 : 0) : what == 2 ? (int)e->runs.size() : -1;
}
void seq_destroy(uint64_t handle) {
  std::lock_guard<std::mutex> g(g_seq_mu);
  auto it = g_seq.find(handle);
  if (it == g_seq.end()) return;
  DeviceCtx& ctx = DeviceCtx::get();
  if (ctx.ready && !ctx.dry) cudaStreamSynchronize(ctx.stream);
  g_seq.erase(it);
}

}  // namespace ag
