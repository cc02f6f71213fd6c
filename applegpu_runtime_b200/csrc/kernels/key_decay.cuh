// What the files of key-decayed matrix states share: the parameters of their kernels, the raw inputs of the convolutions, the
// decay.
#pragma once
#include "common.cuh"
#include "seq_kernels.h"

namespace ag { namespace k {

constexpr int kKdChunk = 32;           // tokens per chunk

struct KdParams {
  const void* proj; const void* a2; const void* g2; const float* bias; const float* rate; const float* conv; const float* norm; const float* beta; const int* pos;
  void* mem; void* y;
  const float* z; const void* gate;      // decay inputs [rows, heads * dim] without bias and gates [rows, heads * vdim], where a product made them
  long long ld, beta_ld, mem_stride, y_ld, gate_ld, ring_off;      // ring_off: bytes from a sequence's memory to its ring
  int n_seq, T, heads, qk_heads, group, dim, vdim, taps, ring, channels;
  int q_off, k_off, v_off, a_off, a_rank, a_ld, g_off, g_rank, g_ld;
  int delta, unit, softplus, gate_silu;
  float inv_tau, q_scale, eps;
  uint8_t* ops; float* u; float* o;      // scratch of the chunk form (u: warp-level scan; o: where a head's values take more than one CTA)
  int chunks, dp;                        // dp: dim padded for the tensor cores
  __device__ float* state(int s) const { return reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(mem) + (long long)s * mem_stride); }
  template <typename T> __device__ T* ring_of(int s) const { return reinterpret_cast<T*>(reinterpret_cast<uint8_t*>(mem) + (long long)s * mem_stride + ring_off); }
};

// Raw input of a channel: `col` its column in proj, `ch` its place among the q | k | v channels, t the token of the portion (negative:
// before it; zero before the sequence's start).
template <typename T>
__device__ __forceinline__ float kd_raw(const KdParams& p, const T* base, const T* ring, int pos, int t, int col, int ch) {
  if (t >= 0) return Cvt<T>::to(base[(long long)t * p.ld + col]);
  const int at = pos + t;
  return at < 0 ? 0.f : Cvt<T>::to(ring[(long long)(at % p.ring) * p.channels + ch]);
}
// One channel at token t behind its convolution and silu, or as it is.
template <typename T>
__device__ __forceinline__ float kd_input(const KdParams& p, const T* base, const T* ring, int pos, int t, int col, int ch) {
  if (p.taps == 0) return Cvt<T>::to(base[(long long)t * p.ld + col]);
  const float* w = p.conv + (long long)ch * p.taps;
  float a = 0.f;
  for (int i = 0; i < p.taps; i++) a = fmaf(__ldg(w + i), kd_raw(p, base, ring, pos, t - (p.taps - 1) + i, col, ch), a);
  return silu_f(a);
}
__device__ __forceinline__ float kd_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float kd_gate(const KdParams& p, float g) { return p.gate_silu ? silu_f(g) : sigmoid_f(g); }

// What the prepare kernel hands to the scan for one chunk of one head. Up to 128 channels (tcgen05 scan): 128-byte swizzled panels of 64
// columns with rows A k (delta rule) and A q, their remainders as further rows; A_32 / A k, then its remainders; one panel of Q, a
// row's remainders behind its high parts; T (delta rule), its remainders as further rows; the chunk's decay and beta in float32.
// Wider (warp-level scan): rows of pitch dp + 8, planes of A q, -W, A_32 / A k, Q, then the decay; U lies beside.
constexpr int kKdAPitch = kKdChunk + 8;
struct KdOpsLayout { int rows1, panels, plane1, plane2, qg, w, kg, q, t, decay, beta, bytes, stride; };     // offsets and sizes in bytes
__host__ __device__ constexpr bool kd_tc(int dp) { return dp <= 128; }
__host__ __device__ constexpr KdOpsLayout kd_ops_layout(int dp, bool delta) {
  KdOpsLayout l{};
  if (kd_tc(dp)) {
    l.rows1 = delta ? 2 * kKdChunk : kKdChunk; l.panels = (dp + 63) / 64;
    l.plane1 = l.rows1 * 128; l.plane2 = l.panels * kKdChunk * 128;      // plane1: from a row to its remainder
    l.qg = delta ? kKdChunk * 128 : 0; l.w = 0; l.kg = l.panels * 2 * l.plane1; l.q = l.kg + 2 * l.plane2; l.t = l.q + kKdChunk * 128;
    l.decay = l.t + (delta ? 2 * kKdChunk * 128 : 0);
  } else {
    l.rows1 = kKdChunk; l.plane1 = l.plane2 = kKdChunk * (dp + 8) * 2;
    l.qg = 0; l.w = 2 * l.plane1; l.kg = l.w + (delta ? 2 * l.plane1 : 0); l.q = l.kg + 2 * l.plane2; l.t = l.decay = l.q + 2 * kKdChunk * kKdAPitch * 2;
  }
  l.beta = l.decay + dp * 4;
  l.bytes = l.beta + kKdChunk * 4;
  l.stride = (l.bytes + 1023) / 1024 * 1024;
  return l;
}

inline int kd_dp(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 96 ? 96 : dim <= 128 ? 128 : dim <= 192 ? 192 : 256; }
// the scan ends with a head's norm and gate where one CTA holds all of its values
inline bool kd_fused(int dp, int vdim) { return kd_tc(dp) && vdim <= 128; }
Status key_decay_chunked_bf16(cudaStream_t s, const KdParams& p);
Status key_decay_chunked_f16(cudaStream_t s, const KdParams& p);

}}  // namespace ag::k
