// Sequence models: decoder-only models described by a list of layers, each a token mixer with its own kind of per-sequence
// memory (a recurrent state, a key cache) beside a feed-forward, run by one engine. See seqmodel.cc.
#pragma once
#include "runtime.h"

namespace ag {

enum class MixerKind : int { Mlstm = 1, LatentAttention = 2, KeyDecay = 3, GroupedAttention = 4 };
enum class LayerForm : int { Parallel = 0, Sequential = 1 };     // see seqmodel.cc
enum KeyDecayFlag : int { kKdDelta = 1, kKdUnit = 2, kKdSoftplus = 4, kKdGateSilu = 8 };

struct SeqLayerCfg {
  MixerKind mixer = MixerKind::Mlstm;
  int heads = 0, dim = 0, vdim = 0;
  int rot_dim = 0, rot_pairs = 0, kv_rank = 0;      // latent attention
  float gate_cap = 0.f;                             // mLSTM
  float score_scale = 0.f;                          // attention
  int kv_heads = 0;                                 // grouped attention, key decay (heads of q and k)
  int window = 0, kv_from = -1;                     // grouped attention: keys a token sees (0: all), layer whose keys it uses (-1: its own)
  float softcap = 0.f;                              // grouped attention
  int taps = 0, a_rank = 0, g_rank = 0, flags = 0;  // key decay (KeyDecayFlag)
  float tau = 1.f;                                  // key decay
  int ff = 0;                                       // 0: no feed-forward
  int glu = 0;                                      // k::Glu
  float ff_limit = 0.f;
};
struct SeqModelCfg {
  int vocab = 0, width = 0;
  float eps = 1e-5f;
  LayerForm form = LayerForm::Parallel;
  float embed_scale = 1.f;
  int loop_start = 0, loop_stop = 0, loop_times = 0;  // loop_times 0: no layer is repeated
  std::vector<SeqLayerCfg> layers;
};
// Weight tensors: embed, head, final norm, step vectors (or an empty record without a loop), then kSeqLayerWeights per layer
// in the order of SeqLayerWeight (empty records where a layer has none).
enum SeqLayerWeight : int { kWNorm1 = 0, kWNorm2, kWIn, kWOut, kWFf, kWAux0, kWAux1, kWAux2, kWPost1, kWPost2, kWDown, kWAux3, kWAux4, kWAux5, kWAux6, kSeqLayerWeights };

Status seq_create(const SeqModelCfg& cfg, const std::vector<TensorRec>& weights, int slots, int max_len, uint64_t* handle);
// The next T tokens of the sequences in slots slot0 .. slot0 + n_seq, all of them of the same portion length. `want`: rows
// (s * T + t) whose logits are asked for; host_logits [n_want, vocab] and picked [n_want] (greedy choice; with one wanted row
// per sequence it also becomes the token seq_decode continues from) may each be null. layers_out: [layer runs, n_seq * T, width].
Status seq_forward(uint64_t handle, int slot0, int n_seq, const int32_t* tokens, int T, const int32_t* want, int n_want, float* host_logits,
                   int32_t* picked, float* layers_out);
// n_steps greedy tokens per sequence, each step one replay of a captured graph (use_graph) -> host_tokens [n_steps, n_seq].
Status seq_decode(uint64_t handle, int slot0, int n_seq, int n_steps, int32_t* host_tokens, bool use_graph);
Status seq_reset(uint64_t handle, int slot, int n);
int seq_length(uint64_t handle, int slot);
int seq_info(uint64_t handle, int what);             // 0 launches of the last decode step, 1 whether it was a graph, 2 layer runs
void seq_destroy(uint64_t handle);

}  // namespace ag
