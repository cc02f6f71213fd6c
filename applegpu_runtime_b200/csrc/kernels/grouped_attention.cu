// Attention of heads that share keys and values in groups, over a cache of normed, turned keys and plain values.
//
//   append  a warp per head and row: RMS norm over the head, the rotation of its first entries (i with i + rot_pairs), queries in
//           place, keys and values into the cache
//   decode  short portions: a cluster per (row, key head), each CTA a split of the keys the row sees, for up to eight query heads
//           at a time; the splits meet over distributed shared memory. Scores, their maximum and the weights are float32.
// Longer portions take prompt_attention straight over the cache.
#include "common.cuh"
#include "seq_kernels.h"
#include "sm100.cuh"
#include <algorithm>

namespace ag { namespace k {

struct GaParams {
  void* proj; const float* q_norm; const float* k_norm; const float2* rot; void* cache; const int* pos; void* y;
  long long ld, seq_stride, y_ld, cld, v_col;
  int n_seq, T, heads, kv_heads, group, dim, vdim, pairs, window, shared, max_len, q_off, k_off, v_off;
  int hg, h_parts;                       // query heads per CTA, CTAs along a group's heads
  float scale, cap, eps;
};

static Status ga_params(const GroupedAttnDesc& d, GaParams* out) {
  if (d.n_seq < 1 || d.T < 1 || d.heads < 1 || d.kv_heads < 1 || d.heads % d.kv_heads || d.dim < 1 || d.vdim < 1 || d.rot_pairs < 0 || 2 * d.rot_pairs > d.dim || d.window < 0)
    return Status::invalid("grouped attention: bad sizes");
  if (!d.proj || !d.cache || !d.pos || !d.q_norm || (!d.shared && !d.k_norm) || (d.rot_pairs && !d.rot_table)) return Status::invalid("grouped attention: missing operand");
  GaParams& p = *out;
  p.proj = d.proj; p.q_norm = d.q_norm; p.k_norm = d.k_norm; p.rot = d.rot_table; p.cache = d.cache; p.pos = d.pos; p.y = d.y;
  p.ld = d.ld; p.seq_stride = d.seq_stride; p.y_ld = d.y_ld; p.cld = grouped_cache_ld(d.kv_heads, d.dim, d.vdim); p.v_col = grouped_v_col(d.kv_heads, d.dim);
  p.n_seq = d.n_seq; p.T = d.T; p.heads = d.heads; p.kv_heads = d.kv_heads; p.group = d.heads / d.kv_heads; p.dim = d.dim; p.vdim = d.vdim; p.pairs = d.rot_pairs;
  p.window = d.window; p.shared = d.shared ? 1 : 0; p.max_len = d.max_len; p.q_off = d.q_off; p.k_off = d.k_off; p.v_off = d.v_off;
  p.scale = d.scale; p.cap = d.softcap; p.eps = d.eps; p.hg = 1; p.h_parts = 1;
  return Status::OK();
}

// ── append ──────────────────────────────────────────────────────────────────
constexpr int kGaThreads = 256;
template <typename T>
__device__ __forceinline__ void ga_norm_turn(const GaParams& p, const T* src, T* dst, const float* w, int position, int lane) {
  float sq = 0.f;
  for (int i = lane; i < p.dim; i += 32) { const float v = Cvt<T>::to(src[i]); sq = fmaf(v, v, sq); }
  const float rs = 1.0f / sqrtf(warp_sum(sq) / (float)p.dim + p.eps);       // also: every lane has read before any writes
  for (int i = lane; i < p.pairs; i += 32) {
    const float2 cs = p.rot[(long long)position * p.pairs + i];
    const float u = Cvt<T>::to(src[i]) * rs * w[i], v = Cvt<T>::to(src[i + p.pairs]) * rs * w[i + p.pairs];
    dst[i] = Cvt<T>::from(u * cs.x - v * cs.y);
    dst[i + p.pairs] = Cvt<T>::from(v * cs.x + u * cs.y);
  }
  for (int i = 2 * p.pairs + lane; i < p.dim; i += 32) dst[i] = Cvt<T>::from(Cvt<T>::to(src[i]) * rs * w[i]);
}
template <typename T>
__global__ void __launch_bounds__(kGaThreads) grouped_append_kernel(const GaParams p) {
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x, s = r / p.T, t = r % p.T, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int position = p.pos[s] + t;
  if (position < 0 || position >= p.max_len) return;
  T* row = reinterpret_cast<T*>(p.proj) + (long long)r * p.ld;
  T* crow = reinterpret_cast<T*>(p.cache) + (long long)s * p.seq_stride + (long long)position * p.cld;
  const int n = p.heads + (p.shared ? 0 : p.kv_heads);
  for (int h = warp; h < n; h += kGaThreads / 32) {
    if (h < p.heads) { T* q = row + p.q_off + (long long)h * p.dim; ga_norm_turn<T>(p, q, q, p.q_norm, position, lane); }
    else { const int g = h - p.heads; ga_norm_turn<T>(p, row + p.k_off + (long long)g * p.dim, crow + (long long)g * p.dim, p.k_norm, position, lane); }
  }
  if (!p.shared) for (int i = threadIdx.x; i < p.kv_heads * p.vdim; i += kGaThreads) crow[p.v_col + i] = row[p.v_off + i];
}
Status grouped_append(cudaStream_t s, const GroupedAttnDesc& d) {
  GaParams p;
  AG_RETURN_IF_ERROR(ga_params(d, &p));
  cudaError_t e = cudaSuccess;
  AG_DISPATCH_FLOAT(d.dtype, T, (e = launch_pdl(grouped_append_kernel<T>, dim3((unsigned)(d.n_seq * d.T)), dim3(kGaThreads), 0, s, p)));
  return cuda_status(e, "grouped append");
}

// ── decode ──────────────────────────────────────────────────────────────────
constexpr int kGdKeys = 64, kGdOut = 8;              // keys per tile; accumulators per thread: heads * vdim <= 256 * kGdOut
static int gd_pitch(int n, size_t esz) { const int per = 16 / (int)esz, q = (n + per - 1) / per; return (q % 2 ? q : q + 1) * per; }   // an odd number of 16-byte pieces

template <typename T, int NO>
__global__ void __launch_bounds__(256) grouped_decode_kernel(const GaParams p, int kp, int vp) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  constexpr int N = Pack<T>::N;
  T* sk = reinterpret_cast<T*>(smem_raw);                          // [kGdKeys][kp]
  T* sv = sk + kGdKeys * kp;                                       // [kGdKeys][vp]
  float* sq = reinterpret_cast<float*>(sv + kGdKeys * vp);         // [hg][kp], zero past dim
  float* sp = sq + p.hg * kp;                                      // [hg][kGdKeys]
  float* s_m = sp + p.hg * kGdKeys;                                // [hg] maximum, sum, rescale factor
  float* s_l = s_m + p.hg;
  float* s_a = s_l + p.hg;
  float* so = s_a + p.hg;                                          // [hg][vdim] of this split
  const int split = (int)sm100::cluster_ctarank(), splits = (int)gridDim.x;
  const int kh = (int)blockIdx.y / p.h_parts, part = (int)blockIdx.y % p.h_parts, h0 = kh * p.group + part * p.hg, nh = min(p.hg, p.group - part * p.hg);
  const int r = blockIdx.z, s = r / p.T, t = r % p.T, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_trigger();
  const int last = min(p.pos[s] + t + 1, p.max_len), from = p.window ? max(0, last - p.window) : 0;
  const int per = ((last - from + splits - 1) / splits + 7) / 8 * 8;
  const int k_lo = min(last, from + split * per), k_hi = min(last, k_lo + per);
  const T* Q = reinterpret_cast<const T*>(p.proj) + (long long)r * p.ld + p.q_off + (long long)h0 * p.dim;
  const T* K = reinterpret_cast<const T*>(p.cache) + (long long)s * p.seq_stride + (long long)kh * p.dim;
  const T* V = reinterpret_cast<const T*>(p.cache) + (long long)s * p.seq_stride + p.v_col + (long long)kh * p.vdim;
  for (int i = threadIdx.x; i < p.hg * kp; i += 256) { const int hh = i / kp, c = i % kp; sq[i] = hh < nh && c < p.dim ? Cvt<T>::to(Q[(long long)hh * p.dim + c]) * p.scale : 0.f; }
  if (threadIdx.x < p.hg) { s_m[threadIdx.x] = -INFINITY; s_l[threadIdx.x] = 0.f; }
  float acc[NO];
#pragma unroll
  for (int n = 0; n < NO; n++) acc[n] = 0.f;
  const int outs = nh * p.vdim;
  const bool kvec = p.dim % N == 0, vvec = p.vdim % N == 0;        // rows of a head then start on 16 bytes
  const int kpacks = (p.dim + N - 1) / N;
  for (int k0 = k_lo; k0 < k_hi; k0 += kGdKeys) {
    const int nk = min(kGdKeys, k_hi - k0);
    __syncthreads();
    auto stage = [&](T* dst, int pitch, const T* src, int n, bool vec) {
      if (vec) {
        const int q = n / N;
        for (int i = threadIdx.x; i < nk * q; i += 256) st16(dst + i / q * pitch + i % q * N, ld16(src + (long long)(k0 + i / q) * p.cld + i % q * N));
      } else {
        const int q = (n + N - 1) / N * N;
        for (int i = threadIdx.x; i < nk * q; i += 256) dst[i / q * pitch + i % q] = i % q < n ? src[(long long)(k0 + i / q) * p.cld + i % q] : Cvt<T>::from(0.f);
      }
    };
    stage(sk, kp, K, p.dim, kvec);
    stage(sv, vp, V, p.vdim, vvec);
    __syncthreads();
    const int key = threadIdx.x & (kGdKeys - 1);
    for (int hh = threadIdx.x / kGdKeys; hh < nh; hh += 256 / kGdKeys) {
      float a = -INFINITY;
      if (key < nk) {
        a = 0.f;
        for (int q = 0; q < kpacks; q++) {
          const Pack<T> kv = *reinterpret_cast<const Pack<T>*>(sk + key * kp + q * N);
          const float* qv = sq + hh * kp + q * N;
#pragma unroll
          for (int e = 0; e < N; e++) a = fmaf(qv[e], Cvt<T>::to(kv.v[e]), a);
        }
        if (p.cap > 0.f) a = p.cap * tanhf(a / p.cap);
      }
      sp[hh * kGdKeys + key] = a;
    }
    __syncthreads();
    for (int hh = warp; hh < nh; hh += 8) {
      const float x0 = sp[hh * kGdKeys + lane], x1 = sp[hh * kGdKeys + lane + 32];
      const float m0 = s_m[hh], m1 = fmaxf(m0, warp_max(fmaxf(x0, x1)));
      const float e0 = x0 == -INFINITY ? 0.f : expf(x0 - m1), e1 = x1 == -INFINITY ? 0.f : expf(x1 - m1);
      const float sum = warp_sum(e0 + e1);
      sp[hh * kGdKeys + lane] = e0; sp[hh * kGdKeys + lane + 32] = e1;
      __syncwarp();
      if (lane == 0) { const float a = m0 == -INFINITY ? 0.f : expf(m0 - m1); s_a[hh] = a; s_l[hh] = s_l[hh] * a + sum; s_m[hh] = m1; }
    }
    __syncthreads();
#pragma unroll
    for (int n = 0; n < NO; n++) {
      const int o = threadIdx.x + n * 256;
      if (o < outs) {
        const int hh = o / p.vdim, c = o % p.vdim;
        float a = acc[n] * s_a[hh];
        const float* w = sp + hh * kGdKeys;
#pragma unroll 8
        for (int j = 0; j < nk; j++) a = fmaf(w[j], Cvt<T>::to(sv[j * vp + c]), a);
        acc[n] = a;
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int n = 0; n < NO; n++) { const int o = threadIdx.x + n * 256; if (o < outs) so[o] = acc[n]; }
  if (splits > 1) sm100::cluster_sync_all(); else __syncthreads();
  // every CTA finishes a share of the outputs
  auto remote = [&](const float* x, int q) {
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(sm100::mapa_u32(sm100::smem_u32(x), (uint32_t)q)));
    return v;
  };
  T* y = reinterpret_cast<T*>(p.y) + (long long)r * p.y_ld + (long long)h0 * p.vdim;
  for (int o = split * 256 + threadIdx.x; o < outs; o += splits * 256) {
    const int hh = o / p.vdim;
    float m = -INFINITY, l = 0.f, a = 0.f;
    for (int q = 0; q < splits; q++) m = fmaxf(m, remote(s_m + hh, q));
    for (int q = 0; q < splits; q++) {
      const float mq = remote(s_m + hh, q);
      if (mq == -INFINITY) continue;
      const float f = expf(mq - m);
      l = fmaf(f, remote(s_l + hh, q), l);
      a = fmaf(f, remote(so + o, q), a);
    }
    y[o] = Cvt<T>::from(a / l);
  }
  if (splits > 1) sm100::cluster_sync_all();        // no CTA leaves while its sums are being read
}

template <typename T, int NO>
static cudaError_t launch_gd(cudaStream_t s, const GaParams& p, int splits, int kp, int vp, size_t smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(grouped_decode_kernel<T, NO>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)splits, (unsigned)(p.kv_heads * p.h_parts), (unsigned)(p.n_seq * p.T)); cfg.blockDim = dim3(256); cfg.dynamicSmemBytes = smem; cfg.stream = s;
  cudaLaunchAttribute at[2];
  at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization; at[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  at[1].id = cudaLaunchAttributeClusterDimension; at[1].val.clusterDim.x = (unsigned)splits; at[1].val.clusterDim.y = 1; at[1].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = 2;
  return cudaLaunchKernelEx(&cfg, grouped_decode_kernel<T, NO>, p, kp, vp);
}

Status grouped_decode(cudaStream_t s, const GroupedAttnDesc& d) {
  GaParams p;
  AG_RETURN_IF_ERROR(ga_params(d, &p));
  if (!d.y || !aligned16(d.cache) || d.seq_stride % 8) return Status::invalid("grouped decode: missing or misaligned operand");
  if (d.vdim > 256 * kGdOut || p.kv_heads > 65535 / p.group || d.n_seq * d.T > 65535) return Status::unsupported("grouped decode: heads too large or too many");
  p.hg = std::min({p.group, 8, 256 * kGdOut / d.vdim});
  p.h_parts = (p.group + p.hg - 1) / p.hg;
  // splits: a cluster of up to eight; about a tile of keys each at least, and no more than fill the machine twice
  const int reach = d.window ? std::min(d.window, d.max_len) : d.max_len;
  int splits = 1;
  while (splits < 8 && splits * 2 * 32 <= reach && splits * p.kv_heads * p.h_parts * d.n_seq * d.T < 2 * sm_count()) splits *= 2;
  cudaError_t e = cudaSuccess;
  AG_DISPATCH_FLOAT(d.dtype, T, {
    const int kp = gd_pitch(d.dim, sizeof(T)), vp = gd_pitch(d.vdim, sizeof(T));
    const size_t smem = (size_t)kGdKeys * (kp + vp) * sizeof(T) + ((size_t)p.hg * kp + (size_t)p.hg * kGdKeys + 3 * p.hg + (size_t)p.hg * d.vdim) * sizeof(float);
    if (smem > 220 * 1024) return Status::unsupported("grouped decode: head too large");
    const int no = (p.hg * d.vdim + 255) / 256;
    if (no <= 1) e = launch_gd<T, 1>(s, p, splits, kp, vp, smem);
    else if (no <= 2) e = launch_gd<T, 2>(s, p, splits, kp, vp, smem);
    else if (no <= 4) e = launch_gd<T, 4>(s, p, splits, kp, vp, smem);
    else e = launch_gd<T, 8>(s, p, splits, kp, vp, smem);
  });
  return cuda_status(e, "grouped decode");
}

}}  // namespace ag::k
