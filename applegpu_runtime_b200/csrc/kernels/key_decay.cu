// Matrix states with one decay per key channel: the token-by-token form and the choice between it and the chunked one.
//
// A CTA works on up to 128 value columns of one head of one sequence (a cluster where a head has more: the head's norm adds their
// sums of squares over distributed shared memory). With r = (diag(a) S)^T k and p = (diag(a) S)^T q taken in one pass over S, the
// rest of a token is u = beta (v - r) (or v), o = p + (k . q) u and the update S <- diag(a) S + k u^T, which is the order of the
// recurrence (o includes what the token itself wrote). S stays in registers from token to token where the CTA's columns fit.
#include "key_decay.cuh"
#include "sm100.cuh"
#include <algorithm>

namespace ag { namespace k {

constexpr int kKsThreads = 512;

// out[i] = sum_r w[row0 + i][r] x[r] for n rows of a [.., ld] matrix: a few lanes per row, 16-byte pieces
template <typename T>
__device__ __forceinline__ void kd_rows(const T* w, int ld, int rank, const float* x, int n, float* out) {
  constexpr int N = Pack<T>::N;
  const int pieces = (rank + N - 1) / N;
  int g = 1;
  while (g < 4 && g * 2 <= pieces) g *= 2;
  const int lane = threadIdx.x % g;
  for (int i0 = 0; i0 < n; i0 += kKsThreads / g) {
    const int i = i0 + (int)threadIdx.x / g;
    float a = 0.f;
    if (i < n) {
      const T* row = w + (long long)i * ld;
#pragma unroll 4
      for (int q = lane; q < pieces; q += g) {
        const Pack<T> v = ld16(row + q * N);
#pragma unroll
        for (int e = 0; e < N; e++) a = fmaf(Cvt<T>::to(v.v[e]), x[q * N + e], a);
      }
    }
    for (int o = g >> 1; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
    if (i < n && lane == 0) out[i] = a;
  }
}
__device__ __forceinline__ void kd_prefetch(const void* at, int bytes) {
  for (int i = threadIdx.x * 128; i < bytes; i += kKsThreads * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const uint8_t*>(at) + i));
}

template <typename T, int VEC, int NR>          // NR rows of S per thread, VEC neighbouring columns of each
__global__ void __launch_bounds__(kKsThreads, VEC * NR <= 32 ? 2 : 1) key_decay_step_kernel(const KdParams p, int slice, int tx_n) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float s_sq[2];
  const int D = p.dim, E = p.vdim, cw = tx_n * VEC;       // cw: columns of a pass
  const int rank = (int)sm100::cluster_ctarank(), n_rank = (int)gridDim.x;
  const int h = blockIdx.y, s = blockIdx.z, qh = h / p.group;
  const int e0 = rank * slice, ne = max(0, min(slice, E - e0));
  const int ty_n = kKsThreads / tx_n, tx = threadIdx.x % tx_n, ty = threadIdx.x / tx_n, lane = threadIdx.x & 31;
  float* part = sm;                      // [2][ty][cw] shares of r and p
  float* s_r = part + 2 * kKsThreads * VEC;      // [2][cw] their sums
  float* sq = s_r + 2 * cw;              // [D] each
  float* sk = sq + D;
  float* sa = sk + D;
  float* sv = sa + D;                    // [slice] each
  float* sg = sv + slice;
  float* so = sg + slice;
  float* sx = so + slice;                // a1 and g1 of the token, padded with zeros to whole packs
  float* sy = sx + p.a_ld;
  // weights start towards the L2 before the previous kernel is waited for
  kd_prefetch(p.bias + h * D, D * 4);
  if (!p.z) kd_prefetch(reinterpret_cast<const T*>(p.a2) + (long long)h * D * p.a_ld, D * p.a_ld * (int)sizeof(T));
  if (!p.gate && p.g_rank) kd_prefetch(reinterpret_cast<const T*>(p.g2) + ((long long)h * E + e0) * p.g_ld, ne * p.g_ld * (int)sizeof(T));
  if (p.taps) {
    const int qk = p.qk_heads * D;
    kd_prefetch(p.conv + (long long)qh * D * p.taps, D * p.taps * 4);
    kd_prefetch(p.conv + (long long)(qk + qh * D) * p.taps, D * p.taps * 4);
    kd_prefetch(p.conv + (long long)(2 * qk + h * E + e0) * p.taps, ne * p.taps * 4);
  }
  pdl_wait();
  pdl_trigger();
  float* S = p.state(s) + (long long)h * D * E + e0;
  const bool resident = slice <= cw;
  float st[NR][VEC];
  const int step = ty_n * E;
  auto load = [&](int c) {
    const float* at = S + ty * E + c;
#pragma unroll
    for (int n = 0; n < NR; n++, at += step) {
      const bool in = n * ty_n + ty < D && c < ne;
      if constexpr (VEC == 4) {
        const float4 f = in ? *reinterpret_cast<const float4*>(at) : make_float4(0.f, 0.f, 0.f, 0.f);
        st[n][0] = f.x; st[n][1] = f.y; st[n][2] = f.z; st[n][3] = f.w;
      } else st[n][0] = in ? *at : 0.f;
    }
  };
  auto store = [&](int c) {
    float* at = S + ty * E + c;
#pragma unroll
    for (int n = 0; n < NR; n++, at += step) {
      if (n * ty_n + ty >= D || c >= ne) continue;
      if constexpr (VEC == 4) *reinterpret_cast<float4*>(at) = make_float4(st[n][0], st[n][1], st[n][2], st[n][3]);
      else *at = st[n][0];
    }
  };
  if (resident) load(tx * VEC);
  const int pos = p.pos[s];
  const T* base = reinterpret_cast<const T*>(p.proj) + (long long)s * p.T * p.ld;
  T* ring = p.ring_of<T>(s);
  const float rate = p.softplus ? p.rate[h] : 0.f;
  for (int t = 0; t < p.T; t++) {
    const T* row = base + (long long)t * p.ld;
    const long long r = (long long)s * p.T + t;
    const float beta_raw = p.delta ? p.beta[r * p.beta_ld + h] : 0.f;
    const int place = p.ring ? (pos + t) % p.ring : 0;            // of this token's raw inputs among the ring's rows
    const bool keep = p.ring && p.T <= kKeyDecayStepTokens;       // nothing of this launch reads the row they take
    __syncthreads();
    for (int i = threadIdx.x; i < 2 * D + ne; i += kKsThreads) {
      const int part_of = i < D ? 0 : i < 2 * D ? 1 : 2;
      const int c = part_of < 2 ? qh * D + i - part_of * D : h * E + e0 + i - 2 * D;
      const int col = (part_of == 0 ? p.q_off : part_of == 1 ? p.k_off : p.v_off) + c, ch = part_of * p.qk_heads * D + c;
      const T raw = row[col];
      float v = Cvt<T>::to(raw);
      if (p.taps) {
        const float* w = p.conv + (long long)ch * p.taps + p.taps - 1;
        v *= __ldg(w);
        for (int b = 1; b < p.taps; b++) {
          float x = 0.f;
          if (t >= b) x = Cvt<T>::to(row[col - (long long)b * p.ld]);
          else if (pos + t >= b) { int q = place - b; if (q < 0) q += p.ring; x = Cvt<T>::to(ring[(long long)q * p.channels + ch]); }
          v = fmaf(__ldg(w - b), x, v);
        }
        v = silu_f(v);
      }
      (part_of == 0 ? sq : part_of == 1 ? sk - D : sv - 2 * D)[i] = v;
      if (keep && (part_of == 2 || (rank == 0 && h % p.group == 0))) ring[(long long)place * p.channels + ch] = raw;
    }
    if (p.z) for (int i = threadIdx.x; i < D; i += kKsThreads) sa[i] = p.z[r * p.heads * D + h * D + i];
    else for (int i = threadIdx.x; i < p.a_ld; i += kKsThreads) sx[i] = i < p.a_rank ? Cvt<T>::to(row[p.a_off + i]) : 0.f;
    if (p.gate || p.g_rank == 0)
      for (int i = threadIdx.x; i < ne; i += kKsThreads)
        sg[i] = p.gate ? Cvt<T>::to(reinterpret_cast<const T*>(p.gate)[r * p.gate_ld + h * E + e0 + i]) : Cvt<T>::to(row[p.g_off + h * E + e0 + i]);
    else for (int i = threadIdx.x; i < p.g_ld; i += kKsThreads) sy[i] = i < p.g_rank ? Cvt<T>::to(row[p.g_off + i]) : 0.f;
    __syncthreads();
    if (!p.z) kd_rows<T>(reinterpret_cast<const T*>(p.a2) + (long long)h * D * p.a_ld, p.a_ld, p.a_rank, sx, D, sa);
    if (!p.gate && p.g_rank) kd_rows<T>(reinterpret_cast<const T*>(p.g2) + ((long long)h * E + e0) * p.g_ld, p.g_ld, p.g_rank, sy, ne, sg);
    // sums over the head, by every warp for itself
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int i = lane; i < D; i += 32) { const float a = sq[i], b = sk[i]; qq = fmaf(a, a, qq); kk = fmaf(b, b, kk); qk = fmaf(a, b, qk); }
    qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
    const float fq = p.unit ? p.q_scale / sqrtf(qq + 1e-6f) : p.q_scale, fk = p.unit ? 1.0f / sqrtf(kk + 1e-6f) : 1.0f;
    qk *= fq * fk;
    const float beta = p.delta ? sigmoid_f(beta_raw) : 1.f;
    __syncthreads();
    for (int i = threadIdx.x; i < D; i += kKsThreads) {
      const float z = sa[i] + p.bias[h * D + i];
      sa[i] = p.softplus ? expf(-rate * kd_softplus(z)) : expf(-kd_softplus(-z) * p.inv_tau);
    }
    __syncthreads();
    for (int c0 = 0; c0 < slice; c0 += cw) {
      const int c = c0 + tx * VEC;
      if (!resident) load(c);
      float rk[VEC], rq[VEC];
#pragma unroll
      for (int v = 0; v < VEC; v++) { rk[v] = 0.f; rq[v] = 0.f; }
#pragma unroll
      for (int n = 0; n < NR; n++) {
        const int d = n * ty_n + ty;
        if (d >= D) break;
        const float a = sa[d], k = sk[d], q = sq[d];
#pragma unroll
        for (int v = 0; v < VEC; v++) { st[n][v] *= a; rk[v] = fmaf(st[n][v], k, rk[v]); rq[v] = fmaf(st[n][v], q, rq[v]); }
      }
      if constexpr (VEC == 4) {
        *reinterpret_cast<float4*>(part + threadIdx.x * 4) = make_float4(rk[0], rk[1], rk[2], rk[3]);
        *reinterpret_cast<float4*>(part + (kKsThreads + threadIdx.x) * 4) = make_float4(rq[0], rq[1], rq[2], rq[3]);
      } else { part[threadIdx.x] = rk[0]; part[kKsThreads + threadIdx.x] = rq[0]; }
      __syncthreads();
      for (int i = threadIdx.x; i < 2 * cw; i += kKsThreads) {
        const float* at = part + (i < cw ? i : kKsThreads * VEC + i - cw);
        float a = 0.f;
#pragma unroll 8
        for (int y = 0; y < ty_n; y++) a += at[y * cw];
        s_r[i] = a * (i < cw ? fk : fq);
      }
      __syncthreads();
      float u[VEC];
#pragma unroll
      for (int v = 0; v < VEC; v++) {
        const float x = c + v < ne ? sv[c + v] : 0.f;
        u[v] = p.delta ? beta * (x - s_r[tx * VEC + v]) : x;
        if (ty == 0 && c + v < ne) so[c + v] = fmaf(qk, u[v], s_r[cw + tx * VEC + v]);
        u[v] *= fk;
      }
#pragma unroll
      for (int n = 0; n < NR; n++) {
        const int d = n * ty_n + ty;
        if (d >= D) break;
        const float k = sk[d];
#pragma unroll
        for (int v = 0; v < VEC; v++) st[n][v] = fmaf(k, u[v], st[n][v]);
      }
      if (!resident) { store(c); __syncthreads(); }
      else if (t + 1 == p.T) store(c);
    }
    __syncthreads();
    float ss = 0.f;
    for (int i = lane; i < ne; i += 32) ss = fmaf(so[i], so[i], ss);
    ss = warp_sum(ss);
    if (n_rank > 1) {
      if (threadIdx.x == 0) s_sq[t & 1] = ss;
      sm100::cluster_sync_all();
      float tot = 0.f;
      for (int q = 0; q < n_rank; q++) {
        float v;
        asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(sm100::mapa_u32(sm100::smem_u32(&s_sq[t & 1]), (uint32_t)q)));
        tot += v;
      }
      ss = tot;
    }
    const float rs = 1.0f / sqrtf(ss / (float)E + p.eps);
    T* y = reinterpret_cast<T*>(p.y) + r * p.y_ld + h * E + e0;
    for (int i = threadIdx.x; i < ne; i += kKsThreads) y[i] = Cvt<T>::from(so[i] * rs * p.norm[e0 + i] * kd_gate(p, sg[i]));
  }
  if (n_rank > 1) sm100::cluster_sync_all();        // no CTA leaves while another may still read its sum
}

// The last taps - 1 raw inputs of a longer portion into the ring.
template <typename T>
__global__ void __launch_bounds__(256) key_decay_tail_kernel(const KdParams p) {
  pdl_wait();
  pdl_trigger();
  const int s = blockIdx.y, keep = min(p.taps - 1, p.T), pos = p.pos[s], qk = p.qk_heads * p.dim;
  T* ring = p.ring_of<T>(s);
  for (int i = blockIdx.x * 256 + threadIdx.x; i < keep * p.channels; i += gridDim.x * 256) {
    const int t = p.T - keep + i / p.channels, ch = i % p.channels;
    const int col = ch < qk ? p.q_off + ch : ch < 2 * qk ? p.k_off + ch - qk : p.v_off + ch - 2 * qk;
    ring[(long long)((pos + t) % p.ring) * p.channels + ch] = reinterpret_cast<const T*>(p.proj)[((long long)s * p.T + t) * p.ld + col];
  }
}

template <typename T, int VEC, int NR>
static cudaError_t launch_ks(cudaStream_t s, const KdParams& p, int ranks, int slice, int tx_n, size_t smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(key_decay_step_kernel<T, VEC, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)ranks, (unsigned)p.heads, (unsigned)p.n_seq); cfg.blockDim = dim3(kKsThreads); cfg.dynamicSmemBytes = smem; cfg.stream = s;
  cudaLaunchAttribute at[2];
  at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization; at[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  at[1].id = cudaLaunchAttributeClusterDimension; at[1].val.clusterDim.x = (unsigned)ranks; at[1].val.clusterDim.y = 1; at[1].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = 2;
  return cudaLaunchKernelEx(&cfg, key_decay_step_kernel<T, VEC, NR>, p, slice, tx_n);
}

static Status key_decay_step(cudaStream_t s, DType dt, const KdParams& p) {
  // four columns a thread where rows of S lie on 16 bytes and a thread's share of them fits its registers
  auto shape = [&](int vec, int* ranks, int* slice, int* tx_n) {
    const int most = 32 * vec;
    *ranks = 1;
    while (*ranks < 8 && (p.vdim + *ranks - 1) / *ranks > most) *ranks *= 2;
    *slice = ((p.vdim + *ranks - 1) / *ranks + vec - 1) / vec * vec;
    *tx_n = 4;
    while (*tx_n < 32 && *tx_n * vec < *slice) *tx_n *= 2;
    return (p.dim + kKsThreads / *tx_n - 1) / (kKsThreads / *tx_n);
  };
  int ranks, slice, tx_n, vec = 4, nr = shape(4, &ranks, &slice, &tx_n);
  if (p.vdim % 4 || nr > 16) { vec = 1; nr = shape(1, &ranks, &slice, &tx_n); }
  const size_t smem = (2 * (size_t)kKsThreads * vec + 2 * (size_t)tx_n * vec + 3 * (size_t)p.dim + 3 * (size_t)slice + p.a_ld + p.g_ld) * sizeof(float);
  if (nr > 32 || smem > 100 * 1024) return Status::unsupported("key decay: head too large");
  cudaError_t e = cudaSuccess;
  AG_DISPATCH_FLOAT(dt, T, {
    if (vec == 4) e = nr <= 2 ? launch_ks<T, 4, 2>(s, p, ranks, slice, tx_n, smem) : nr <= 4 ? launch_ks<T, 4, 4>(s, p, ranks, slice, tx_n, smem)
                    : nr <= 8 ? launch_ks<T, 4, 8>(s, p, ranks, slice, tx_n, smem) : launch_ks<T, 4, 16>(s, p, ranks, slice, tx_n, smem);
    else e = nr <= 8 ? launch_ks<T, 1, 8>(s, p, ranks, slice, tx_n, smem) : launch_ks<T, 1, 32>(s, p, ranks, slice, tx_n, smem);
  });
  return cuda_status(e, "key decay step");
}

// Scratch of a portion longer than kKeyDecayStepTokens: z, the gates, and for the chunk form what its kernels hand on.
struct KdWork { float* z; void* gate; uint8_t* ops; float* u; float* o; size_t total; };
static KdWork kd_layout(const KeyDecayDesc& d, void* base) {
  KdWork w = {};
  uint8_t* p = static_cast<uint8_t*>(base);
  size_t o = 0;
  auto take = [&](size_t bytes) { uint8_t* r = p + o; o += (bytes + 255) / 256 * 256; return r; };
  const size_t rows = (size_t)d.n_seq * d.T;
  w.z = reinterpret_cast<float*>(take(rows * d.heads * d.dim * sizeof(float)));
  w.gate = d.g_rank ? take(rows * pad8((int64_t)d.heads * d.vdim) * dtype_size(d.dtype)) : nullptr;
  if (key_decay_chunk_eligible(d)) {
    const size_t n = (size_t)d.n_seq * d.heads * ((d.T + kKdChunk - 1) / kKdChunk);
    w.ops = take(n * kd_ops_layout(kd_dp(d.dim), d.delta).stride);
    if (!kd_tc(kd_dp(d.dim))) w.u = reinterpret_cast<float*>(take(n * d.vdim * kKdChunk * sizeof(float)));
    if (!kd_fused(kd_dp(d.dim), d.vdim)) w.o = reinterpret_cast<float*>(take(rows * d.heads * d.vdim * sizeof(float)));
  }
  w.total = o;
  return w;
}
size_t key_decay_work_bytes(const KeyDecayDesc& d) { return d.T <= kKeyDecayStepTokens ? 0 : kd_layout(d, nullptr).total; }

bool key_decay_chunk_eligible(const KeyDecayDesc& d) {
  return (d.dtype == DType::BF16 || d.dtype == DType::F16) && d.T > kKeyDecayStepTokens && d.dim <= 256 && !d.simple && matmul_status_word() != nullptr;
}

Status key_decay(cudaStream_t s, const KeyDecayDesc& d, int* launches) {
  if (d.n_seq < 1 || d.T < 1 || d.heads < 1 || d.qk_heads < 1 || d.heads % d.qk_heads || d.dim < 1 || d.vdim < 1 || d.a_rank < 1 || d.g_rank < 0 || d.taps < 0)
    return Status::invalid("key decay: bad sizes");
  if (!d.proj || !d.a2 || !d.bias || !d.norm || !d.mem || !d.pos || !d.y || (d.taps && !d.conv) || (d.softplus && !d.rate) || (d.delta && !d.beta) || (d.g_rank && !d.g2) ||
      d.mem_stride % 16 || !aligned16(d.mem) || !aligned16(d.a2) || !aligned16(d.g2))
    return Status::invalid("key decay: missing or misaligned operand");
  if (d.heads > 65535 || d.n_seq > 65535) return Status::unsupported("key decay: too many heads or sequences for one launch");
  KdParams p = {};
  p.proj = d.proj; p.a2 = d.a2; p.g2 = d.g2; p.bias = d.bias; p.rate = d.rate; p.conv = d.conv; p.norm = d.norm; p.beta = d.beta; p.pos = d.pos; p.mem = d.mem; p.y = d.y;
  p.ld = d.ld; p.beta_ld = d.beta_ld; p.mem_stride = d.mem_stride; p.y_ld = d.y_ld; p.ring_off = (long long)key_decay_state_bytes(d.heads, d.dim, d.vdim);
  p.n_seq = d.n_seq; p.T = d.T; p.heads = d.heads; p.qk_heads = d.qk_heads; p.group = d.heads / d.qk_heads; p.dim = d.dim; p.vdim = d.vdim; p.taps = d.taps;
  p.ring = key_decay_ring(d.taps); p.channels = key_decay_channels(d.heads, d.qk_heads, d.dim, d.vdim);
  p.q_off = d.q_off; p.k_off = d.k_off; p.v_off = d.v_off; p.a_off = d.a_off; p.a_rank = d.a_rank; p.a_ld = (int)pad8(d.a_rank); p.g_off = d.g_off; p.g_rank = d.g_rank;
  p.g_ld = (int)pad8(d.g_rank);
  p.delta = d.delta; p.unit = d.unit; p.softplus = d.softplus; p.gate_silu = d.gate_silu; p.inv_tau = 1.0f / d.tau; p.q_scale = d.q_scale; p.eps = d.eps;
  if (d.T <= kKeyDecayStepTokens) { *launches += 1; return key_decay_step(s, d.dtype, p); }
  if (!d.work) return Status::invalid("key decay: no workspace");
  const KdWork w = kd_layout(d, d.work);
  const size_t esz = dtype_size(d.dtype);
  auto product = [&](int off, int rank, const void* wt, int n, void* out, int64_t out_ld, bool f32) {
    GemmDesc g;
    g.dtype = d.dtype; g.b_dtype = d.dtype; g.a = static_cast<const uint8_t*>(d.proj) + (size_t)off * esz; g.b = wt; g.c = out; g.m = (int64_t)d.n_seq * d.T; g.n = n; g.k = rank; g.batch = 1;
    g.a_row = d.ld; g.a_col = 1; g.a_batch = 0; g.b_row = 1; g.b_col = pad8(rank); g.b_batch = 0; g.c_row = out_ld; g.c_batch = 0;
    g.c_f32 = f32 && d.dtype != DType::F32;
    *launches += 1;
    return matmul(s, g);
  };
  AG_RETURN_IF_ERROR(product(d.a_off, d.a_rank, d.a2, d.heads * d.dim, w.z, (int64_t)d.heads * d.dim, true));
  p.z = w.z;
  if (d.g_rank) {
    p.gate_ld = pad8((int64_t)d.heads * d.vdim);
    AG_RETURN_IF_ERROR(product(d.g_off, d.g_rank, d.g2, d.heads * d.vdim, w.gate, p.gate_ld, false));
    p.gate = w.gate;
  }
  if (w.ops) {
    p.chunks = (d.T + kKdChunk - 1) / kKdChunk; p.dp = kd_dp(d.dim); p.ops = w.ops; p.u = w.u; p.o = w.o;
    *launches += kd_fused(p.dp, p.vdim) ? 2 : 3;
    AG_RETURN_IF_ERROR(d.dtype == DType::BF16 ? key_decay_chunked_bf16(s, p) : key_decay_chunked_f16(s, p));
  } else {
    *launches += 1;
    AG_RETURN_IF_ERROR(key_decay_step(s, d.dtype, p));
  }
  if (p.ring) {
    *launches += 1;
    cudaError_t e = cudaSuccess;
    const unsigned blocks = (unsigned)std::min(64, (p.channels * (p.taps - 1) + 255) / 256);
    AG_DISPATCH_FLOAT(d.dtype, T, (e = launch_pdl(key_decay_tail_kernel<T>, dim3(blocks, (unsigned)d.n_seq), dim3(256), 0, s, p)));
    return cuda_status(e, "key decay: convolution inputs");
  }
  return Status::OK();
}

}}  // namespace ag::k
