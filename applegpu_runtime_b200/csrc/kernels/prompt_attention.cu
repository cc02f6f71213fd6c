// Attention of a prompt portion over cached or expanded keys and values: the form on CUDA cores, float32 arithmetic, any sizes.
// Heads may share keys and values in groups, keys may end in a part that all heads share, scores may be capped, and a row may
// see a window of the last keys only. prompt_attention_tc.cu has the tensor-core form.
#include "common.cuh"
#include "seq_kernels.h"

namespace ag { namespace k {

struct PaParams {
  const void* q; const void* k; const void* v; const void* kr; void* y;
  long long q_ld, k_ld, v_ld, kr_ld, y_ld, q_b, k_b, v_b, kr_b, y_b;
  int T, past, heads, group, dim, rot, vdim, window;
  float scale, cap;
};
template <typename T, int TQ>
__global__ void __launch_bounds__(256) prompt_attention_kernel(const PaParams p) {
  extern __shared__ __align__(16) float sm[];
  const int D = p.dim + p.rot, E = p.vdim;
  float* sq = sm;                        // [TQ][D]
  float* sk = sq + TQ * D;               // [TQ][D + 1]
  float* sv = sk + TQ * (D + 1);         // [TQ][E]
  float* so = sv + TQ * E;               // [TQ][E]
  float* sp = so + TQ * E;               // [TQ][TQ + 1]
  float* s_m = sp + TQ * (TQ + 1);       // [TQ] running maximum, sum, rescale factor
  float* s_l = s_m + TQ;
  float* s_a = s_l + TQ;
  pdl_wait();
  pdl_trigger();
  const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * TQ, h = blockIdx.y;     // longest rows first
  const int rows = min(TQ, p.T - q0);
  const long long b = blockIdx.z;
  const T* Q = reinterpret_cast<const T*>(p.q) + b * p.q_b + (long long)h * D;
  const int kh = h / p.group;
  const T* K = reinterpret_cast<const T*>(p.k) + b * p.k_b + (long long)kh * p.dim;
  const T* V = reinterpret_cast<const T*>(p.v) + b * p.v_b + (long long)kh * E;
  const T* KR = reinterpret_cast<const T*>(p.kr) + b * p.kr_b;
  for (int i = threadIdx.x; i < TQ * D; i += 256) {
    const int t = i / D;
    sq[i] = t < rows ? Cvt<T>::to(Q[(long long)(q0 + t) * p.q_ld + i % D]) * p.scale : 0.f;
  }
  for (int i = threadIdx.x; i < TQ * E; i += 256) so[i] = 0.f;
  if (threadIdx.x < TQ) { s_m[threadIdx.x] = -INFINITY; s_l[threadIdx.x] = 0.f; }
  const int n_keys = p.past + q0 + rows;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int first = p.window ? max(0, p.past + q0 - p.window + 1) : 0;     // of the tile's first row
  for (int k0 = first; k0 < n_keys; k0 += TQ) {
    const int nk = min(TQ, n_keys - k0);
    __syncthreads();
    for (int i = threadIdx.x; i < nk * D; i += 256) {
      const int j = i / D, c = i % D;
      sk[j * (D + 1) + c] = c < p.dim ? Cvt<T>::to(K[(long long)(k0 + j) * p.k_ld + c]) : Cvt<T>::to(KR[(long long)(k0 + j) * p.kr_ld + c - p.dim]);
    }
    for (int i = threadIdx.x; i < nk * E; i += 256) sv[i] = Cvt<T>::to(V[(long long)(k0 + i / E) * p.v_ld + i % E]);
    __syncthreads();
    for (int i = threadIdx.x; i < TQ * TQ; i += 256) {
      const int t = i / TQ, j = i % TQ;
      float v = -INFINITY;
      const int back = p.past + q0 + t - (k0 + j);
      if (t < rows && j < nk && back >= 0 && (!p.window || back < p.window)) {
        v = 0.f;
        for (int c = 0; c < D; c++) v = fmaf(sq[t * D + c], sk[j * (D + 1) + c], v);
        if (p.cap > 0.f) v = p.cap * tanhf(v / p.cap);
      }
      sp[t * (TQ + 1) + j] = v;
    }
    __syncthreads();
    for (int t = warp; t < rows; t += 8) {
      const float v = lane < TQ ? sp[t * (TQ + 1) + lane] : -INFINITY;
      const float m1 = fmaxf(s_m[t], warp_max(v));
      const float e = v == -INFINITY ? 0.f : expf(v - m1);
      const float sum = warp_sum(e);
      if (lane < TQ) sp[t * (TQ + 1) + lane] = e;
      __syncwarp();
      if (lane == 0) {
        const float a = m1 == -INFINITY ? 1.f : expf(s_m[t] - m1);
        s_a[t] = a; s_l[t] = s_l[t] * a + sum; s_m[t] = m1;
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < rows * E; i += 256) {
      const int t = i / E, e = i % E;
      float a = so[i] * s_a[t];
      for (int j = 0; j < nk; j++) a = fmaf(sp[t * (TQ + 1) + j], sv[j * E + e], a);
      so[i] = a;
    }
  }
  __syncthreads();
  T* Y = reinterpret_cast<T*>(p.y) + b * p.y_b + (long long)h * E;
  for (int i = threadIdx.x; i < rows * E; i += 256) Y[(long long)(q0 + i / E) * p.y_ld + i % E] = Cvt<T>::from(so[i] / s_l[i / E]);
}

template <typename T, int TQ>
static cudaError_t launch_pa(cudaStream_t s, const PaParams& p, int n_seq, size_t smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(prompt_attention_kernel<T, TQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  return launch_pdl(prompt_attention_kernel<T, TQ>, dim3((unsigned)((p.T + TQ - 1) / TQ), (unsigned)p.heads, (unsigned)n_seq), dim3(256), smem, s, p);
}

Status prompt_attention(cudaStream_t s, const PromptAttnDesc& d) {
  if (d.T < 1 || d.past < 0 || d.heads < 1 || d.heads > 65535 || d.dim < 1 || d.rot_dim < 0 || d.vdim < 1 || !d.q || !d.k || !d.v || (d.rot_dim && !d.k_rot) || !d.y || d.group < 1 || d.window < 0 || d.n_seq < 1 || d.n_seq > 65535)
    return Status::invalid("prompt attention: bad description");
  if (prompt_attention_tc_eligible(d)) return prompt_attention_tc(s, d);
  PaParams p;
  p.q = d.q; p.k = d.k; p.v = d.v; p.kr = d.k_rot; p.y = d.y; p.q_ld = d.q_ld; p.k_ld = d.k_ld; p.v_ld = d.v_ld; p.kr_ld = d.k_rot_ld; p.y_ld = d.y_ld;
  p.q_b = d.q_b; p.k_b = d.k_b; p.v_b = d.v_b; p.kr_b = d.k_rot_b; p.y_b = d.y_b;
  p.T = d.T; p.past = d.past; p.heads = d.heads; p.dim = d.dim; p.rot = d.rot_dim; p.vdim = d.vdim; p.group = d.group; p.window = d.window; p.scale = d.scale; p.cap = d.softcap;
  auto smem = [&](int tq) { return ((size_t)tq * (2 * (d.dim + d.rot_dim) + 1) + 2 * (size_t)tq * d.vdim + (size_t)tq * (tq + 1) + 3 * tq) * sizeof(float); };
  const size_t lim = 220 * 1024;
  if (smem(8) > lim) return Status::unsupported("prompt attention: head too large");
  cudaError_t e = cudaSuccess;
  AG_DISPATCH_FLOAT(d.dtype, T, (e = smem(32) <= lim ? launch_pa<T, 32>(s, p, d.n_seq, smem(32)) : smem(16) <= lim ? launch_pa<T, 16>(s, p, d.n_seq, smem(16)) : launch_pa<T, 8>(s, p, d.n_seq, smem(8))));
  return cuda_status(e, "prompt attention");
}

}}  // namespace ag::k
