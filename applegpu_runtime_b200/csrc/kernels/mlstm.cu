// mLSTM: a matrix memory per head with scalar, exponentially gated input and forget gates.
//
// With i_t, f_t the log gates of a token and m_t = max(f_t + m_{t-1}, i_t) the running maximum that keeps every factor
// below one, the state after token t is S_t = sum_j w_tj k_j v_j^T + r_t S_0 (n_t the same with k alone), where
//     F_t = f_1 + .. + f_t,   w_tj = exp(F_t - F_j + i_j - m_t),   r_t = exp(F_t + m_0 - m_t).
// A prompt portion therefore splits into chunks that can be worked on side by side:
//   gates    F_t and m_t for all tokens: a scan with (F, M) o (F', M') = (F + F', max(M + F', M')), in double precision,
//            so that the differences F_t - F_j of far apart tokens lose nothing
//   chunk    what a chunk adds to the state when it starts from zero
//   carry    the state in front of every chunk, from the one before it; the last one is the sequence's new state
//   output   o_t = (q_t S_c) r_t + sum over the chunk's j <= t of w_tj (q_t k_j) v_j, the normaliser alike, the division
//            by max(|n q|, exp(-m)) + 1e-6, the head's RMS norm, its weight and the output gate
// A generated token (and a portion of a few) takes mlstm_step instead, which updates the state in place.
#include "mlstm.cuh"
#include "sm100.cuh"

namespace ag { namespace k {

size_t mlstm_work_bytes(int n_seq, int T, int heads, int dim, int vdim) {
  size_t total = 0;
  ml_layout(nullptr, n_seq, T, heads, dim, vdim, &total);
  return total;
}

// ── gates ───────────────────────────────────────────────────────────────────
__global__ void __launch_bounds__(256) ml_gates_kernel(const MlParams p) {
  __shared__ double sF[8], sM[8];
  __shared__ double cF, cM;
  pdl_wait();
  pdl_trigger();
  const int sh = blockIdx.x, s = sh / p.heads, h = sh % p.heads;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* mp = p.m_of(s) + h;
  const float bi = p.gate_bias[h], bf = p.gate_bias[p.heads + h];
  if (threadIdx.x == 0) { cF = 0.0; cM = (double)*mp; p.w.m_start[(long long)sh * (p.w.chunks + 1)] = *mp; }
  __syncthreads();
  for (int t0 = 0; t0 < p.T; t0 += 256) {
    const int t = t0 + threadIdx.x;
    double F = 0.0, M = -1e300;
    float li = 0.f;
    if (t < p.T) {
      const float* g = p.gates + ((long long)s * p.T + t) * p.gates_ld;
      li = ml_cap(g[h] + bi, p.cap);
      F = (double)ml_log_sigmoid(ml_cap(g[p.heads + h] + bf, p.cap));
      M = (double)li;
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double Fp = __shfl_up_sync(0xffffffffu, F, o), Mp = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) { M = fmax(Mp + F, M); F += Fp; }
    }
    if (lane == 31) { sF[warp] = F; sM[warp] = M; }
    __syncthreads();
    double bF = cF, bM = cM;                          // what lies before this warp
    for (int w = 0; w < warp; w++) { bM = fmax(bM + sF[w], sM[w]); bF += sF[w]; }
    const double bF0 = cF;                            // the chunk starts here: 256 threads, 256 tokens
    M = fmax(bM + F, M);
    F += bF;
    if (t < p.T) {
      const long long o = (long long)sh * p.T + t;
      constexpr double kLog2e = 1.4426950408889634;
      const double a = (F - bF0) * kLog2e, b = (double)li * kLog2e - a;
      float4 ab;
      ab.x = (float)a; ab.y = (float)(a - (double)ab.x); ab.z = (float)b; ab.w = (float)(b - (double)ab.z);
      p.w.ab[o] = ab;
      p.w.m2[o] = (float)(M * kLog2e);
      p.w.F[o] = F; p.w.log_i[o] = li; p.w.m[o] = (float)M;
      if ((t + 1) % kMlChunk == 0 || t + 1 == p.T) p.w.m_start[(long long)sh * (p.w.chunks + 1) + (t + kMlChunk) / kMlChunk] = (float)M;
      if (t + 1 == p.T) *mp = (float)M;
    }
    __syncthreads();
    if (threadIdx.x == 255) { cF = F; cM = M; }       // past the end F and M carry on unchanged (f = 0, i = -inf)
    __syncthreads();
  }
}

// ── chunk: the state a chunk builds up from zero ────────────────────────────
constexpr int kMlCd = 32, kMlCe = 64, kMlCt = 32;     // rows and columns of the state per CTA, tokens per pass
template <typename T>
__global__ void __launch_bounds__(256) ml_chunk_kernel(const MlParams p) {
  __shared__ float ks[kMlCt][kMlCd + 1];
  __shared__ float vs[kMlCt][kMlCe + 4];
  pdl_wait();
  pdl_trigger();
  const int tiles_e = (p.vdim + kMlCe - 1) / kMlCe;
  const int d0 = (int)blockIdx.x / tiles_e * kMlCd, e0 = (int)blockIdx.x % tiles_e * kMlCe;
  const int c = blockIdx.y, sh = blockIdx.z, s = sh / p.heads, h = sh % p.heads;
  const int t0 = c * kMlChunk, t1 = min(p.T, t0 + kMlChunk);
  const double* F = p.w.F + (long long)sh * p.T;
  const float* li = p.w.log_i + (long long)sh * p.T;
  const double F_end = F[t1 - 1];
  const float m_end = p.w.m[(long long)sh * p.T + t1 - 1];
  const T* base = reinterpret_cast<const T*>(p.proj) + (long long)s * p.T * p.ld;
  const int kq = p.heads * p.dim, koff = kq + h * p.dim, voff = 2 * kq + h * p.vdim;
  const int ee = threadIdx.x & 63, dg = threadIdx.x >> 6;   // a thread: one column, eight rows
  float acc[8], nacc = 0.f;
#pragma unroll
  for (int i = 0; i < 8; i++) acc[i] = 0.f;
  for (int t = t0; t < t1; t += kMlCt) {
    for (int i = threadIdx.x; i < kMlCt * kMlCd; i += 256) {
      const int tt = i / kMlCd, dd = i % kMlCd;
      float v = 0.f;
      if (t + tt < t1 && d0 + dd < p.dim)
        v = Cvt<T>::to(base[(long long)(t + tt) * p.ld + koff + d0 + dd]) * expf((float)(F_end - F[t + tt]) + li[t + tt] - m_end);
      ks[tt][dd] = v;
    }
    for (int i = threadIdx.x; i < kMlCt * kMlCe; i += 256) {
      const int tt = i / kMlCe, e = i % kMlCe;
      vs[tt][e] = (t + tt < t1 && e0 + e < p.vdim) ? Cvt<T>::to(base[(long long)(t + tt) * p.ld + voff + e0 + e]) : 0.f;
    }
    __syncthreads();
#pragma unroll 4
    for (int tt = 0; tt < kMlCt; tt++) {
      const float v = vs[tt][ee];
#pragma unroll
      for (int i = 0; i < 8; i++) acc[i] = fmaf(ks[tt][dg * 8 + i], v, acc[i]);
    }
    if (e0 == 0 && threadIdx.x < kMlCd)
      for (int tt = 0; tt < kMlCt; tt++) nacc += ks[tt][threadIdx.x];
    __syncthreads();
  }
  const long long ci = (long long)sh * p.w.chunks + c;
  float* S = p.w.S + ci * p.dim * p.vdim;
#pragma unroll
  for (int i = 0; i < 8; i++) {
    const int dd = d0 + dg * 8 + i;
    if (dd < p.dim && e0 + ee < p.vdim) S[(long long)dd * p.vdim + e0 + ee] = acc[i];
  }
  if (e0 == 0 && threadIdx.x < kMlCd && d0 + threadIdx.x < p.dim) p.w.n[ci * p.dim + d0 + threadIdx.x] = nacc;
}

// ── carry: the chunks' own states become the states in front of them ────────
// A thread owns VEC neighbouring elements of a head's S (or one of n, by the blocks past S).
template <typename T, int VEC>      // T: storage type of the planes the tensor-core output kernel reads; float: none, the states stay float32
__global__ void __launch_bounds__(256) ml_carry_kernel(const MlParams p, int s_blocks) {
  __shared__ float s_decay[256];
  pdl_wait();
  pdl_trigger();
  const int sh = blockIdx.y, s = sh / p.heads, h = sh % p.heads;
  const long long n_state = (long long)p.dim * p.vdim;
  const double* F = p.w.F + (long long)sh * p.T;
  const float* ms = p.w.m_start + (long long)sh * (p.w.chunks + 1);
  const bool is_n = (int)blockIdx.x >= s_blocks;
  const long long i = is_n ? ((long long)(blockIdx.x - s_blocks) * 256 + threadIdx.x) : ((long long)blockIdx.x * 256 + threadIdx.x) * VEC;
  const bool live = i < (is_n ? p.dim : n_state);
  float* home = is_n ? p.n_of(s) + (long long)h * p.dim + i : p.S_of(s) + h * n_state + i;
  float* own = is_n ? p.w.n + (long long)sh * p.w.chunks * p.dim + i : p.w.S + (long long)sh * p.w.chunks * n_state + i;
  const long long step = is_n ? p.dim : n_state;
  float v[VEC];
  auto load = [&](const float* q, float (&o)[VEC]) {
    if constexpr (VEC == 4) {
      if (!is_n) { const float4 f = *reinterpret_cast<const float4*>(q); o[0] = f.x; o[1] = f.y; o[2] = f.z; o[3] = f.w; return; }
    }
    o[0] = q[0];
  };
  auto store = [&](float* q, const float (&o)[VEC]) {
    if constexpr (VEC == 4) {
      if (!is_n) { *reinterpret_cast<float4*>(q) = make_float4(o[0], o[1], o[2], o[3]); return; }
    }
    q[0] = o[0];
  };
#pragma unroll
  for (int e = 0; e < VEC; e++) v[e] = 0.f;
  if (live) load(home, v);
  for (int c0 = 0; c0 < p.w.chunks; c0 += 256) {
    const int nc = min(256, p.w.chunks - c0);
    __syncthreads();
    if ((int)threadIdx.x < nc) {
      const int c = c0 + threadIdx.x, t1 = min(p.T, (c + 1) * kMlChunk);
      const double Fc = F[t1 - 1] - (c ? F[c * kMlChunk - 1] : 0.0);
      s_decay[threadIdx.x] = expf((float)Fc + ms[c] - ms[c + 1]);
    }
    __syncthreads();
    if (!live) continue;
#pragma unroll 4
    for (int k = 0; k < nc; k++) {
      const int c = c0 + k;
      float u[VEC];
#pragma unroll
      for (int e = 0; e < VEC; e++) u[e] = 0.f;
      load(own + c * step, u);
      if (sizeof(T) == 4 || is_n) store(own + c * step, v);
      else {
        T* plane = reinterpret_cast<T*>(p.w.planes) + ((long long)sh * p.w.chunks + c) * 2 * n_state + i;
        alignas(8) T hi[VEC], lo[VEC];
#pragma unroll
        for (int e = 0; e < VEC; e++) { hi[e] = Cvt<T>::from(v[e]); lo[e] = Cvt<T>::from(v[e] - Cvt<T>::to(hi[e])); }
        if constexpr (VEC * sizeof(T) == 8) { *reinterpret_cast<uint2*>(plane) = *reinterpret_cast<const uint2*>(hi); *reinterpret_cast<uint2*>(plane + n_state) = *reinterpret_cast<const uint2*>(lo); }
        else {
#pragma unroll
          for (int e = 0; e < VEC; e++) { plane[e] = hi[e]; plane[n_state + e] = lo[e]; }
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; e++) v[e] = fmaf(v[e], s_decay[k], u[e]);
    }
  }
  if (live) store(home, v);
}

// ── output ──────────────────────────────────────────────────────────────────
// One CTA: TQ rows of one head. The state in front of the chunk takes part as `dim` more keys whose "scores" are
// q * r_t and whose values are the rows of S.
template <typename T, int TQ>
__global__ void __launch_bounds__(256) ml_output_kernel(const MlParams p) {
  extern __shared__ __align__(16) float sm[];
  const int D = p.dim, E = p.vdim;
  float* sq = sm;                          // [TQ][D]
  float* sk = sq + TQ * D;                 // [TQ][D + 1]
  float* sv = sk + TQ * (D + 1);           // [TQ][E]
  float* so = sv + TQ * E;                 // [TQ][E]
  float* sp = so + TQ * E;                 // [TQ][TQ + 1]
  float* sn = sp + TQ * (TQ + 1);          // [TQ] n . q
  pdl_wait();
  pdl_trigger();
  const int q0 = blockIdx.x * TQ, h = blockIdx.y, s = blockIdx.z, sh = s * p.heads + h;
  const int rows = min(TQ, p.T - q0);
  const int c = q0 / kMlChunk, t0 = c * kMlChunk;
  const T* base = reinterpret_cast<const T*>(p.proj) + (long long)s * p.T * p.ld;
  const int kq = p.heads * D, qoff = h * D, koff = kq + h * D, voff = 2 * kq + h * E, goff = 2 * kq + p.heads * E + h * E;
  const double* F = p.w.F + (long long)sh * p.T;
  const float* li = p.w.log_i + (long long)sh * p.T;
  const float* m = p.w.m + (long long)sh * p.T;
  const double F_c = c ? F[t0 - 1] : 0.0;
  const float m_c = p.w.m_start[(long long)sh * (p.w.chunks + 1) + c];
  const float* S = p.w.S + ((long long)sh * p.w.chunks + c) * D * E;
  const float* n = p.w.n + ((long long)sh * p.w.chunks + c) * D;
  for (int i = threadIdx.x; i < TQ * D; i += 256) {
    const int t = i / D;
    sq[i] = t < rows ? Cvt<T>::to(base[(long long)(q0 + t) * p.ld + qoff + i % D]) * p.q_scale : 0.f;
  }
  for (int i = threadIdx.x; i < TQ * E; i += 256) so[i] = 0.f;
  if (threadIdx.x < TQ) sn[threadIdx.x] = 0.f;
  __syncthreads();
  auto accumulate = [&](int keys) {         // so += sp x sv
    for (int i = threadIdx.x; i < TQ * E; i += 256) {
      const int t = i / E, e = i % E;
      float a = so[i];
      for (int j = 0; j < keys; j++) a = fmaf(sp[t * (TQ + 1) + j], sv[j * E + e], a);
      so[i] = a;
    }
  };
  for (int d0 = 0; d0 < D; d0 += TQ) {      // what lies in front of the chunk
    const int nd = min(TQ, D - d0);
    for (int i = threadIdx.x; i < nd * E; i += 256) sv[i] = S[(long long)d0 * E + i];
    for (int i = threadIdx.x; i < TQ * TQ; i += 256) {
      const int t = i / TQ, j = i % TQ;
      float v = 0.f;
      if (t < rows && j < nd) v = sq[t * D + d0 + j] * expf((float)(F[q0 + t] - F_c) + m_c - m[q0 + t]);
      sp[t * (TQ + 1) + j] = v;
    }
    __syncthreads();
    if (threadIdx.x < TQ) {
      float a = sn[threadIdx.x];
      for (int j = 0; j < nd; j++) a = fmaf(sp[threadIdx.x * (TQ + 1) + j], n[d0 + j], a);
      sn[threadIdx.x] = a;
    }
    accumulate(nd);
    __syncthreads();
  }
  for (int k0 = t0; k0 < q0 + rows; k0 += TQ) {
    const int nk = min(TQ, q0 + rows - k0);
    for (int i = threadIdx.x; i < nk * D; i += 256) sk[i / D * (D + 1) + i % D] = Cvt<T>::to(base[(long long)(k0 + i / D) * p.ld + koff + i % D]);
    for (int i = threadIdx.x; i < nk * E; i += 256) sv[i] = Cvt<T>::to(base[(long long)(k0 + i / E) * p.ld + voff + i % E]);
    __syncthreads();
    for (int i = threadIdx.x; i < TQ * TQ; i += 256) {
      const int t = i / TQ, j = i % TQ;
      float v = 0.f;
      if (t < rows && j < nk && k0 + j <= q0 + t) {
        for (int dd = 0; dd < D; dd++) v = fmaf(sq[t * D + dd], sk[j * (D + 1) + dd], v);
        v *= expf((float)(F[q0 + t] - F[k0 + j]) + li[k0 + j] - m[q0 + t]);
      }
      sp[t * (TQ + 1) + j] = v;
    }
    __syncthreads();
    if (threadIdx.x < TQ) {
      float a = sn[threadIdx.x];
      for (int j = 0; j < nk; j++) a += sp[threadIdx.x * (TQ + 1) + j];
      sn[threadIdx.x] = a;
    }
    accumulate(nk);
    __syncthreads();
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int t = warp; t < rows; t += 8) {
    const float den = 1.0f / (fmaxf(fabsf(sn[t]), expf(-m[q0 + t])) + 1e-6f);
    float sqs = 0.f;
    for (int e = lane; e < E; e += 32) { const float v = so[t * E + e] * den; so[t * E + e] = v; sqs = fmaf(v, v, sqs); }
    const float rs = 1.0f / sqrtf(warp_sum(sqs) / (float)E + p.eps);
    const T* g = base + (long long)(q0 + t) * p.ld + goff;
    T* y = reinterpret_cast<T*>(p.y) + ((long long)s * p.T + q0 + t) * p.y_ld + h * E;
    for (int e = lane; e < E; e += 32) y[e] = Cvt<T>::from(so[t * E + e] * rs * p.norm[h * E + e] * sigmoid_f(Cvt<T>::to(g[e])));
  }
}

static size_t ml_output_smem(int tq, int dim, int vdim) { return ((size_t)tq * dim + (size_t)tq * (dim + 1) + 2 * (size_t)tq * vdim + (size_t)tq * (tq + 1) + tq) * sizeof(float); }

template <typename T, int TQ>
static cudaError_t launch_ml_output(cudaStream_t s, const MlParams& p, size_t smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(ml_output_kernel<T, TQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  return launch_pdl(ml_output_kernel<T, TQ>, dim3((unsigned)((p.T + TQ - 1) / TQ), (unsigned)p.heads, (unsigned)p.n_seq), dim3(256), smem, s, p);
}

static Status ml_params(const MlstmDesc& d, MlParams* out) {
  if (d.n_seq < 1 || d.T < 1 || d.heads < 1 || d.dim < 1 || d.vdim < 1 || !d.proj || !d.gates || !d.state || !d.y || !d.gate_bias || !d.norm)
    return Status::invalid("mlstm: bad description");
  MlParams& p = *out;
  p.proj = d.proj; p.gates = d.gates; p.gate_bias = d.gate_bias; p.norm = d.norm; p.state = d.state; p.y = d.y;
  p.ld = d.ld; p.gates_ld = d.gates_ld; p.state_stride = d.state_stride; p.y_ld = d.y_ld;
  p.n_seq = d.n_seq; p.T = d.T; p.heads = d.heads; p.dim = d.dim; p.vdim = d.vdim; p.cap = d.gate_cap; p.eps = d.eps;
  p.q_scale = (float)(1.0 / sqrt((double)d.dim));
  p.w = MlWork{};
  return Status::OK();
}

Status mlstm_prefill(cudaStream_t s, const MlstmDesc& d) {
  MlParams p;
  AG_RETURN_IF_ERROR(ml_params(d, &p));
  if (!d.work) return Status::invalid("mlstm: no workspace");
  p.w = ml_layout(d.work, d.n_seq, d.T, d.heads, d.dim, d.vdim, nullptr);
  const int sh = d.n_seq * d.heads;
  if (sh > 65535 || p.w.chunks > 65535) return Status::unsupported("mlstm: too many heads or chunks for one launch");
  cudaError_t e = launch_pdl(ml_gates_kernel, dim3((unsigned)sh), dim3(256), 0, s, p);
  if (e != cudaSuccess) return cuda_status(e, "mlstm gates");
  const bool tc = !d.simple && mlstm_tc_eligible(d);
  if (tc) {
    AG_RETURN_IF_ERROR(mlstm_chunk_tc(s, d.dtype, p));
  } else {
    const int tiles = (d.dim + kMlCd - 1) / kMlCd * ((d.vdim + kMlCe - 1) / kMlCe);
    AG_DISPATCH_FLOAT(d.dtype, T, (e = launch_pdl(ml_chunk_kernel<T>, dim3((unsigned)tiles, (unsigned)p.w.chunks, (unsigned)sh), dim3(256), 0, s, p)));
    if (e != cudaSuccess) return cuda_status(e, "mlstm chunk states");
  }
  const bool vec = d.vdim % 4 == 0 && d.state_stride % 4 == 0 && aligned16(d.state);
  const int s_blocks = (int)(((long long)d.dim * d.vdim + 256 * (vec ? 4 : 1) - 1) / (256 * (vec ? 4 : 1)));
  const dim3 cgrid((unsigned)(s_blocks + (d.dim + 255) / 256), (unsigned)sh);
  auto carry = [&](auto tag) {
    using T = decltype(tag);
    return vec ? launch_pdl(ml_carry_kernel<T, 4>, cgrid, dim3(256), 0, s, p, s_blocks) : launch_pdl(ml_carry_kernel<T, 1>, cgrid, dim3(256), 0, s, p, s_blocks);
  };
  e = !tc ? carry(0.f) : d.dtype == DType::BF16 ? carry(__nv_bfloat16()) : carry(__half());
  if (e != cudaSuccess) return cuda_status(e, "mlstm carry");
  if (tc) return mlstm_output_tc(s, d.dtype, p);
  const size_t lim = 220 * 1024;
  const size_t s32 = ml_output_smem(32, d.dim, d.vdim), s16 = ml_output_smem(16, d.dim, d.vdim), s8 = ml_output_smem(8, d.dim, d.vdim);
  if (s8 > lim) return Status::unsupported("mlstm: head too large");
  AG_DISPATCH_FLOAT(d.dtype, T, (e = s32 <= lim ? launch_ml_output<T, 32>(s, p, s32) : s16 <= lim ? launch_ml_output<T, 16>(s, p, s16) : launch_ml_output<T, 8>(s, p, s8)));
  return cuda_status(e, "mlstm output");
}

// ── token by token ──────────────────────────────────────────────────────────
// A cluster works on one head of one sequence, each CTA on a slice of the value columns of S; the head's RMS norm adds
// the slices' sums of squares over distributed shared memory. S stays in global memory and is read and written once per
// token, by the same thread.
constexpr int kMsThreads = 256;
template <typename T, int VEC>
__global__ void __launch_bounds__(kMsThreads) ml_step_kernel(const MlParams p, int slice, int tx_n) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[33];
  __shared__ float s_sq[2];
  __shared__ float s_keep, s_write, s_m;
  const int D = p.dim, E = p.vdim;
  const int rank = (int)sm100::cluster_ctarank(), n_rank = (int)gridDim.x;
  const int h = blockIdx.y, s = blockIdx.z;
  const int e0 = rank * slice, ne = max(0, min(slice, E - e0));
  float* sq = sm;                       // [D]
  float* sk = sq + D;                   // [D]
  float* sn = sk + D;                   // [D]
  float* sv = sn + D;                   // [slice]
  float* so = sv + slice;               // [slice]
  float* part = so + ((slice + 3) / 4 * 4 - slice) + slice;   // [ty][slice]
  const int ty_n = kMsThreads / tx_n, tx = threadIdx.x % tx_n, ty = threadIdx.x / tx_n;
  pdl_wait();
  pdl_trigger();
  float* S = p.S_of(s) + (long long)h * D * E + e0;
  float* n = p.n_of(s) + (long long)h * D;
  float* mp = p.m_of(s) + h;
  const T* base = reinterpret_cast<const T*>(p.proj) + (long long)s * p.T * p.ld;
  const int kq = p.heads * D, qoff = h * D, koff = kq + h * D, voff = 2 * kq + h * E + e0, goff = 2 * kq + p.heads * E + h * E + e0;
  for (int i = threadIdx.x; i < D; i += kMsThreads) sn[i] = n[i];
  if (threadIdx.x == 0) s_m = *mp;
  for (int t = 0; t < p.T; t++) {
    const T* row = base + (long long)t * p.ld;
    __syncthreads();
    if (threadIdx.x == 0) {
      const float* g = p.gates + ((long long)s * p.T + t) * p.gates_ld;
      const float li = ml_cap(g[h] + p.gate_bias[h], p.cap);
      const float lf = ml_log_sigmoid(ml_cap(g[p.heads + h] + p.gate_bias[p.heads + h], p.cap));
      const float m1 = fmaxf(lf + s_m, li);
      s_keep = expf(lf + s_m - m1); s_write = expf(li - m1); s_m = m1;
    }
    for (int i = threadIdx.x; i < D; i += kMsThreads) { sq[i] = Cvt<T>::to(row[qoff + i]) * p.q_scale; sk[i] = Cvt<T>::to(row[koff + i]); }
    for (int i = threadIdx.x; i < ne; i += kMsThreads) sv[i] = Cvt<T>::to(row[voff + i]);
    __syncthreads();
    const float keep = s_keep, write = s_write;
    float nq = 0.f;
    for (int i = threadIdx.x; i < D; i += kMsThreads) {
      const float v = fmaf(keep, sn[i], write * sk[i]);
      sn[i] = v;
      nq = fmaf(v, sq[i], nq);
    }
    nq = block_sum(nq, red);
    for (int c = tx * VEC; c < ne; c += tx_n * VEC) {
      float a[VEC], v[VEC];
#pragma unroll
      for (int j = 0; j < VEC; j++) { a[j] = 0.f; v[j] = sv[c + j] * write; }
#pragma unroll 8
      for (int dd = ty; dd < D; dd += ty_n) {
        float* q = S + (long long)dd * E + c;
        float st[VEC];
        if constexpr (VEC == 4) { const float4 f = *reinterpret_cast<const float4*>(q); st[0] = f.x; st[1] = f.y; st[2] = f.z; st[3] = f.w; }
        else st[0] = q[0];
#pragma unroll
        for (int j = 0; j < VEC; j++) { st[j] = fmaf(keep, st[j], sk[dd] * v[j]); a[j] = fmaf(st[j], sq[dd], a[j]); }
        if constexpr (VEC == 4) *reinterpret_cast<float4*>(q) = make_float4(st[0], st[1], st[2], st[3]);
        else q[0] = st[0];
      }
#pragma unroll
      for (int j = 0; j < VEC; j++) part[ty * slice + c + j] = a[j];
    }
    __syncthreads();
    const float den = 1.0f / (fmaxf(fabsf(nq), expf(-s_m)) + 1e-6f);
    float ss = 0.f;
    for (int e = threadIdx.x; e < ne; e += kMsThreads) {
      float o = 0.f;
      for (int y = 0; y < ty_n; y++) o += part[y * slice + e];
      o *= den;
      so[e] = o;
      ss = fmaf(o, o, ss);
    }
    ss = block_sum(ss, red);
    if (n_rank > 1) {
      if (threadIdx.x == 0) s_sq[t & 1] = ss;
      sm100::cluster_sync_all();
      float tot = 0.f;
      for (int r = 0; r < n_rank; r++) {
        float v;
        asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(sm100::mapa_u32(sm100::smem_u32(&s_sq[t & 1]), (uint32_t)r)));
        tot += v;
      }
      ss = tot;
    }
    const float rs = 1.0f / sqrtf(ss / (float)E + p.eps);
    T* y = reinterpret_cast<T*>(p.y) + ((long long)s * p.T + t) * p.y_ld + h * E + e0;
    for (int e = threadIdx.x; e < ne; e += kMsThreads) y[e] = Cvt<T>::from(so[e] * rs * p.norm[h * E + e0 + e] * sigmoid_f(Cvt<T>::to(row[goff + e])));
  }
  if (n_rank > 1) sm100::cluster_sync_all();        // no CTA leaves while another may still read its sum
  if (rank == 0) {
    __syncthreads();
    for (int i = threadIdx.x; i < D; i += kMsThreads) n[i] = sn[i];
    if (threadIdx.x == 0) *mp = s_m;
  }
}

template <typename T, int VEC>
static cudaError_t launch_ml_step(cudaStream_t s, const MlParams& p, int ranks, int slice, int tx_n, size_t smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(ml_step_kernel<T, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)ranks, (unsigned)p.heads, (unsigned)p.n_seq); cfg.blockDim = dim3(kMsThreads); cfg.dynamicSmemBytes = smem; cfg.stream = s;
  cudaLaunchAttribute attr2[2];
  attr2[0].id = cudaLaunchAttributeProgrammaticStreamSerialization; attr2[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  attr2[1].id = cudaLaunchAttributeClusterDimension; attr2[1].val.clusterDim.x = (unsigned)ranks; attr2[1].val.clusterDim.y = 1; attr2[1].val.clusterDim.z = 1;
  cfg.attrs = attr2; cfg.numAttrs = 2;
  return cudaLaunchKernelEx(&cfg, ml_step_kernel<T, VEC>, p, slice, tx_n);
}

Status mlstm_step(cudaStream_t s, const MlstmDesc& d) {
  MlParams p;
  AG_RETURN_IF_ERROR(ml_params(d, &p));
  if (d.heads > 65535 || d.n_seq > 65535) return Status::unsupported("mlstm: too many heads for one launch");
  const bool vec = d.vdim % 4 == 0 && d.state_stride % 4 == 0 && aligned16(d.state);
  int ranks = 1;
  while (ranks < 8 && d.vdim / (ranks * 2) >= 16) ranks *= 2;
  int slice = (d.vdim + ranks - 1) / ranks;
  if (vec) slice = (slice + 3) / 4 * 4;
  int tx_n = 1;
  while (tx_n < 32 && tx_n * (vec ? 4 : 1) < slice) tx_n *= 2;
  const size_t smem = (3 * (size_t)d.dim + 2 * (size_t)slice + 8 + (size_t)(kMsThreads / tx_n) * slice) * sizeof(float);
  if (smem > 200 * 1024) return Status::unsupported("mlstm: head too large");
  cudaError_t e = cudaSuccess;
  AG_DISPATCH_FLOAT(d.dtype, T, (e = vec ? launch_ml_step<T, 4>(s, p, ranks, slice, tx_n, smem) : launch_ml_step<T, 1>(s, p, ranks, slice, tx_n, smem)));
  return cuda_status(e, "mlstm step");
}

}}  // namespace ag::k
