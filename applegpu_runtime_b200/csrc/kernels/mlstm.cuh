// What the two files of mLSTM kernels share: the chunk length, the scratch of a portion, the parameters of its kernels.
#pragma once
#include "common.cuh"
#include "seq_kernels.h"

namespace ag { namespace k {

constexpr int kMlChunk = 256;          // tokens per chunk

__device__ __forceinline__ float ml_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float ml_cap(float z, float cap) { return cap * tanhf(z / cap); }

// Scratch of a portion. F, log_i, m are [n_seq * heads, T]; m_start [n_seq * heads, chunks + 1]; states and normalisers of
// the chunks [n_seq * heads, chunks, ...]. For the tensor-core kernels also, per token, (a, b) with F_t - F_c = a and i - a = b in
// log2 units, each as a float and its remainder, the running maximum in log2 units, and the states in front of the chunks as
// 16-bit planes (high part, remainder): planes [n_seq * heads, chunks, 2, dim, vdim].
struct MlWork {
  double* F; float* log_i; float* m; float* m_start; float* S; float* n; float4* ab; float* m2; uint16_t* planes;
  int chunks;
};
inline size_t ml_align(size_t v) { return (v + 255) / 256 * 256; }
inline MlWork ml_layout(void* base, int n_seq, int T, int heads, int dim, int vdim, size_t* total) {
  MlWork w;
  const size_t sh = (size_t)n_seq * heads;
  w.chunks = (T + kMlChunk - 1) / kMlChunk;
  uint8_t* p = static_cast<uint8_t*>(base);
  size_t o = 0;
  auto take = [&](size_t bytes) { uint8_t* r = p + o; o += ml_align(bytes); return r; };
  w.F = reinterpret_cast<double*>(take(sh * T * sizeof(double)));
  w.log_i = reinterpret_cast<float*>(take(sh * T * sizeof(float)));
  w.m = reinterpret_cast<float*>(take(sh * T * sizeof(float)));
  w.m_start = reinterpret_cast<float*>(take(sh * (w.chunks + 1) * sizeof(float)));
  w.S = reinterpret_cast<float*>(take(sh * w.chunks * (size_t)dim * vdim * sizeof(float)));
  w.n = reinterpret_cast<float*>(take(sh * w.chunks * (size_t)dim * sizeof(float)));
  w.ab = reinterpret_cast<float4*>(take(sh * T * sizeof(float4)));
  w.m2 = reinterpret_cast<float*>(take(sh * T * sizeof(float)));
  w.planes = reinterpret_cast<uint16_t*>(take(sh * w.chunks * 2 * (size_t)dim * vdim * sizeof(uint16_t)));
  if (total) *total = o;
  return w;
}

struct MlParams {
  const void* proj; const float* gates; const float* gate_bias; const float* norm; float* state; void* y;
  long long ld, gates_ld, state_stride, y_ld;
  int n_seq, T, heads, dim, vdim;
  float cap, eps, q_scale;
  MlWork w;
  __device__ float* S_of(int s) const { return state + (long long)s * state_stride; }
  __device__ float* n_of(int s) const { return S_of(s) + (long long)heads * dim * vdim; }
  __device__ float* m_of(int s) const { return n_of(s) + (long long)heads * dim; }
};

// Tensor-core forms of the chunk and output kernels (mlstm_tc.cu).
bool mlstm_tc_eligible(const MlstmDesc& d);
Status mlstm_chunk_tc(cudaStream_t s, DType dt, const MlParams& p);
Status mlstm_output_tc(cudaStream_t s, DType dt, const MlParams& p);

}}  // namespace ag::k
