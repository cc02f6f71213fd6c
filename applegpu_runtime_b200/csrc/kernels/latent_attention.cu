// Latent attention: keys and values of all heads are linear images of one normed latent per token, plus one rotated
// key part shared by the heads; the cache holds only those two.
//
//   append    one row per CTA: rotates the query parts, norms the latent, rotates the key part, writes the cache row
//   prefill   prompt_attention over keys and values expanded from the cache (the GEMM that expands them is the caller's)
//   decode    short portions stay in the latent space: W_uk is applied to the query instead of to every key, W_uv to the
//             attended latent instead of to every value, so that a step reads each cached row once for all heads.
//             prepare -> attend over splits of the keys -> merge the splits and apply W_uv.
// Scores, their maximum and the weights are float32 throughout.
#include "common.cuh"
#include "seq_kernels.h"
#include "mma_sync.cuh"

namespace ag { namespace k {

struct LaParams {
  void* proj; const float* c_norm; const float2* rot; void* cache; const int* pos; const void* uk; const void* uv; void* y;
  long long ld, seq_stride, w_ld, y_ld;
  int n_seq, T, heads, dim, rot_dim, vdim, rank, pairs, max_len, cld, coff;   // cld: cache pitch, coff: column of the rotated part
  float scale, eps;
  float* q_eff; float* part; int splits;
};

static Status la_params(const LatentDesc& d, LaParams* out) {
  if (d.n_seq < 1 || d.T < 1 || d.heads < 1 || d.dim < 1 || d.rot_dim < 0 || d.vdim < 1 || d.kv_rank < 1 || 2 * d.rot_pairs > d.rot_dim)
    return Status::invalid("latent attention: bad sizes");
  if (!d.proj || !d.cache || !d.pos || !d.c_norm || (d.rot_pairs && !d.rot_table)) return Status::invalid("latent attention: missing operand");
  LaParams& p = *out;
  p.proj = d.proj; p.c_norm = d.c_norm; p.rot = d.rot_table; p.cache = d.cache; p.pos = d.pos; p.uk = d.w_uk; p.uv = d.w_uv; p.y = d.y;
  p.ld = d.ld; p.seq_stride = d.seq_stride; p.w_ld = d.w_ld; p.y_ld = d.y_ld;
  p.n_seq = d.n_seq; p.T = d.T; p.heads = d.heads; p.dim = d.dim; p.rot_dim = d.rot_dim; p.vdim = d.vdim; p.rank = d.kv_rank; p.pairs = d.rot_pairs;
  p.max_len = d.max_len; p.cld = (int)latent_cache_ld(d.kv_rank, d.rot_dim); p.coff = (int)pad8(d.kv_rank);
  p.scale = d.scale; p.eps = d.eps; p.q_eff = nullptr; p.part = nullptr; p.splits = 1;
  return Status::OK();
}

// The latent and the rotated key part of one row into its cache row (whole block).
template <typename T>
__device__ __forceinline__ void la_cache_row(const LaParams& p, const T* row, T* crow, int position, float* red) {
  const T* c = row + (long long)p.heads * (p.dim + p.rot_dim);
  const T* kr = c + p.rank;
  T* dst = crow + p.coff;
  constexpr int KEEP = 8;                                // values of the latent a thread keeps (the rest is read again)
  float keep[KEEP], sq = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; k++) { const int i = threadIdx.x + k * blockDim.x; keep[k] = i < p.rank ? Cvt<T>::to(c[i]) : 0.f; }
  for (int i = threadIdx.x; i < p.pairs; i += blockDim.x) {
    const float2 cs = p.rot[(long long)position * p.pairs + i];
    const float u = Cvt<T>::to(kr[2 * i]), v = Cvt<T>::to(kr[2 * i + 1]);
    dst[2 * i] = Cvt<T>::from(u * cs.x - v * cs.y);
    dst[2 * i + 1] = Cvt<T>::from(v * cs.x + u * cs.y);
  }
#pragma unroll
  for (int k = 0; k < KEEP; k++) sq = fmaf(keep[k], keep[k], sq);
  for (int i = threadIdx.x + KEEP * blockDim.x; i < p.rank; i += blockDim.x) { const float v = Cvt<T>::to(c[i]); sq = fmaf(v, v, sq); }
  const float rs = 1.0f / sqrtf(block_sum(sq, red) / (float)p.rank + p.eps);
#pragma unroll
  for (int k = 0; k < KEEP; k++) { const int i = threadIdx.x + k * blockDim.x; if (i < p.rank) crow[i] = Cvt<T>::from(keep[k] * rs * p.c_norm[i]); }
  for (int i = threadIdx.x + KEEP * blockDim.x; i < p.rank; i += blockDim.x) crow[i] = Cvt<T>::from(Cvt<T>::to(c[i]) * rs * p.c_norm[i]);
  for (int i = 2 * p.pairs + threadIdx.x; i < p.rot_dim; i += blockDim.x) dst[i] = kr[i];
}

constexpr int kLaThreads = 128;
template <typename T>
__global__ void __launch_bounds__(kLaThreads) latent_append_kernel(const LaParams p) {
  __shared__ float red[33];
  pdl_wait();
  pdl_trigger();
  const int r = blockIdx.x, s = r / p.T, t = r % p.T;
  const int position = p.pos[s] + t;
  if (position < 0 || position >= p.max_len) return;
  T* row = reinterpret_cast<T*>(p.proj) + (long long)r * p.ld;
  T* crow = reinterpret_cast<T*>(p.cache) + (long long)s * p.seq_stride + (long long)position * p.cld;
  // a warp per head, a lane per pair (read and written as one word when pairs lie on words), four heads in flight
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, hd = p.dim + p.rot_dim;
  constexpr int HF = 4, HW = kLaThreads / 32;
  const bool words = sizeof(T) == 2 && p.dim % 2 == 0 && hd % 2 == 0 && (reinterpret_cast<uintptr_t>(row) & 3u) == 0;
  for (int j = lane; j < p.pairs; j += 32) {
    const float2 cs = p.rot[(long long)position * p.pairs + j];
    T* q0 = row + p.dim + 2 * j;
    for (int h0 = warp; h0 < p.heads; h0 += HW * HF) {
      alignas(8) T t[HF][2];
#pragma unroll
      for (int k = 0; k < HF; k++) {
        const int h = h0 + HW * k;
        if (h >= p.heads) continue;
        const T* q = q0 + (long long)h * hd;
        if (words) *reinterpret_cast<uint32_t*>(t[k]) = *reinterpret_cast<const uint32_t*>(q); else { t[k][0] = q[0]; t[k][1] = q[1]; }
      }
#pragma unroll
      for (int k = 0; k < HF; k++) {
        const int h = h0 + HW * k;
        if (h >= p.heads) continue;
        T* q = q0 + (long long)h * hd;
        const float u = Cvt<T>::to(t[k][0]), v = Cvt<T>::to(t[k][1]);
        t[k][0] = Cvt<T>::from(u * cs.x - v * cs.y);
        t[k][1] = Cvt<T>::from(v * cs.x + u * cs.y);
        if (words) *reinterpret_cast<uint32_t*>(q) = *reinterpret_cast<const uint32_t*>(t[k]); else { q[0] = t[k][0]; q[1] = t[k][1]; }
      }
    }
  }
  la_cache_row<T>(p, row, crow, position, red);
}

Status latent_append(cudaStream_t s, const LatentDesc& d) {
  LaParams p;
  AG_RETURN_IF_ERROR(la_params(d, &p));
  cudaError_t e = cudaSuccess;
  AG_DISPATCH_FLOAT(d.dtype, T, (e = launch_pdl(latent_append_kernel<T>, dim3((unsigned)(d.n_seq * d.T)), dim3(kLaThreads), 0, s, p)));
  return cuda_status(e, "latent append");
}

// ── decode ──────────────────────────────────────────────────────────────────
// prepare: CTA h < heads: the query of head h in cache-row coordinates, scaled: (q W_uk | 0 | rotated part | 0); CTA `heads`
// appends the row to the cache.
template <typename T>
__global__ void __launch_bounds__(256) latent_decode_prepare_kernel(const LaParams p) {
  extern __shared__ __align__(16) float sq[];            // [dim]
  __shared__ float red[33];
  const int h = blockIdx.x, r = blockIdx.y, s = r / p.T, t = r % p.T;
  pdl_wait();
  pdl_trigger();
  const int position = p.pos[s] + t;
  if (position < 0 || position >= p.max_len) return;
  const T* row = reinterpret_cast<const T*>(p.proj) + (long long)r * p.ld;
  if (h == p.heads) {
    la_cache_row<T>(p, row, reinterpret_cast<T*>(p.cache) + (long long)s * p.seq_stride + (long long)position * p.cld, position, red);
    return;
  }
  const T* q = row + (long long)h * (p.dim + p.rot_dim);
  float* out = p.q_eff + ((long long)r * p.heads + h) * p.cld;
  for (int i = threadIdx.x; i < p.dim; i += 256) sq[i] = Cvt<T>::to(q[i]);
  for (int i = threadIdx.x; i < p.cld - p.coff; i += 256) {
    float v = 0.f;
    if (i < 2 * p.pairs) {
      const float2 cs = p.rot[(long long)position * p.pairs + i / 2];
      const float a = Cvt<T>::to(q[p.dim + (i & ~1)]), b = Cvt<T>::to(q[p.dim + (i | 1)]);
      v = (i & 1) ? b * cs.x + a * cs.y : a * cs.x - b * cs.y;
    } else if (i < p.rot_dim) v = Cvt<T>::to(q[p.dim + i]);
    out[p.coff + i] = v * p.scale;
  }
  __syncthreads();
  // 16-byte pieces of the rows of W_uk: a thread owns one piece's columns and every G-th row, the G partial sums meet in
  // shared memory
  constexpr int N = Pack<T>::N;
  const T* uk = reinterpret_cast<const T*>(p.uk) + (long long)h * p.dim * p.w_ld;
  float* part = sq + p.dim;
  const int nv = p.coff / N, G = nv >= 256 ? 1 : 256 / nv, g = threadIdx.x / nv, col = threadIdx.x % nv;
  if (g < G) {
    float a[N];
#pragma unroll
    for (int e = 0; e < N; e++) a[e] = 0.f;
#pragma unroll 8
    for (int d = g; d < p.dim; d += G) {
      const Pack<T> w = ld16(uk + (long long)d * p.w_ld + col * N);
      const float x = sq[d];
#pragma unroll
      for (int e = 0; e < N; e++) a[e] = fmaf(x, Cvt<T>::to(w.v[e]), a[e]);
    }
#pragma unroll
    for (int e = 0; e < N; e++) part[g * p.coff + col * N + e] = a[e];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < p.coff; i += 256) {
    float a = 0.f;
    for (int k = 0; k < G; k++) a += part[k * p.coff + i];
    out[i] = i < p.rank ? a * p.scale : 0.f;
  }
}

// attend: CTA = (split of the keys, eight heads, row); a warp per head. Lane = key for the scores, lanes across the latent
// for the weighted sum. Leaves (maximum, sum, unnormalised latent) per split.
constexpr int kLdKeys = 32, kLdHeads = 8;
template <typename T, int NR>
__global__ void __launch_bounds__(256) latent_decode_attend_kernel(const LaParams p) {
  extern __shared__ __align__(16) float sm[];
  constexpr int PADE = sizeof(T) == 4 ? 1 : 2;           // keeps the row pitch an odd number of 32-bit words
  const int cp = p.cld + PADE;
  float* sq = sm;                                        // [kLdHeads][cld]
  T* sk = reinterpret_cast<T*>(sq + kLdHeads * p.cld);   // [kLdKeys][cp]
  const int split = blockIdx.x, r = blockIdx.z, s = r / p.T, t = r % p.T;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = (int)blockIdx.y * kLdHeads + warp;
  pdl_wait();
  pdl_trigger();
  const int n_keys = min(p.pos[s] + t + 1, p.max_len);
  const int per = ((n_keys + p.splits - 1) / p.splits + kLdKeys - 1) / kLdKeys * kLdKeys;
  const int k_lo = split * per, k_hi = min(n_keys, k_lo + per);
  const bool live = h < p.heads;
  for (int i = threadIdx.x; i < kLdHeads * p.cld; i += 256) {
    const int hh = (int)blockIdx.y * kLdHeads + i / p.cld;
    sq[i] = hh < p.heads && k_lo < k_hi ? p.q_eff[((long long)r * p.heads + hh) * p.cld + i % p.cld] : 0.f;
  }
  float m = -INFINITY, l = 0.f, o[NR];
#pragma unroll
  for (int j = 0; j < NR; j++) o[j] = 0.f;
  const T* cache = reinterpret_cast<const T*>(p.cache) + (long long)s * p.seq_stride;
  constexpr int N = Pack<T>::N;
  const float* qh = sq + warp * p.cld;
  for (int k0 = k_lo; k0 < k_hi; k0 += kLdKeys) {
    const int nk = min(kLdKeys, k_hi - k0);
    __syncthreads();
    for (int i = threadIdx.x; i < nk * (p.cld / N); i += 256) {
      const int j = i / (p.cld / N), c = i % (p.cld / N) * N;
      const Pack<T> v = ld16(cache + (long long)(k0 + j) * p.cld + c);
      uint32_t* dst = reinterpret_cast<uint32_t*>(sk + j * cp + c);
      const uint32_t* src = reinterpret_cast<const uint32_t*>(&v);
      dst[0] = src[0]; dst[1] = src[1]; dst[2] = src[2]; dst[3] = src[3];
    }
    __syncthreads();
    if (!live) continue;
    float sc = -INFINITY;
    if (lane < nk) {
      const T* kr = sk + lane * cp;
      float a0 = 0.f, a1 = 0.f;
      for (int c = 0; c < p.rank; c += 2) {
        a0 = fmaf(qh[c], Cvt<T>::to(kr[c]), a0);
        if (c + 1 < p.rank) a1 = fmaf(qh[c + 1], Cvt<T>::to(kr[c + 1]), a1);
      }
      for (int c = p.coff; c < p.coff + p.rot_dim; c += 2) {
        a0 = fmaf(qh[c], Cvt<T>::to(kr[c]), a0);
        if (c + 1 < p.coff + p.rot_dim) a1 = fmaf(qh[c + 1], Cvt<T>::to(kr[c + 1]), a1);
      }
      sc = a0 + a1;
    }
    const float m1 = fmaxf(m, warp_max(sc));
    const float e = lane < nk ? expf(sc - m1) : 0.f;
    const float a = m == -INFINITY ? 0.f : expf(m - m1);
    l = l * a + warp_sum(e);
    m = m1;
#pragma unroll
    for (int j = 0; j < NR; j++) o[j] *= a;
    for (int key = 0; key < nk; key++) {
      const float w = __shfl_sync(0xffffffffu, e, key);
      const T* kr = sk + key * cp;
#pragma unroll
      for (int j = 0; j < NR; j++) {
        const int c = lane + 32 * j;
        if (c < p.rank) o[j] = fmaf(w, Cvt<T>::to(kr[c]), o[j]);
      }
    }
  }
  if (!live) return;
  float* dst = p.part + (((long long)r * p.heads + h) * p.splits + split) * (p.rank + 2);
  if (lane == 0) { dst[0] = m; dst[1] = l; }
#pragma unroll
  for (int j = 0; j < NR; j++) {
    const int c = lane + 32 * j;
    if (c < p.rank) dst[2 + c] = o[j];
  }
}

// The same on tensor cores for 16-bit caches: CTA = (split, sixteen heads, row), blocks of 64 keys in shared memory. The query
// (float32) and the weights (float32) enter the products as high part and remainder. A warp takes 8 keys of the scores and
// every eighth 8-column tile of the latent; each warp's two heads get their maximum, weights and sum in between.
constexpr int kLmKeys = 64, kLmHeads = 16;
__host__ __device__ inline int lm_k(int cld) { return (cld + 31) / 32 * 32; }
__host__ __device__ inline int lm_pitch(int cld) { const int p = lm_k(cld) / 8; return (p % 2 ? p : p + 1) * 8; }   // odd number of 16-byte pieces: no bank conflicts
static size_t lm_smem(int cld) { return ((size_t)kLmKeys + 2 * kLmHeads) * lm_pitch(cld) * 2 + (size_t)kLmHeads * (kLmKeys + 1) * 4 + 2 * (size_t)kLmHeads * (kLmKeys + 8) * 2 + 4 * kLmHeads * 4; }
template <typename T, int NW>          // NW: 8-column latent tiles per warp, rank <= 64 * NW
__global__ void __launch_bounds__(256) latent_decode_attend_mma_kernel(const LaParams p) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int K = lm_k(p.cld), P = lm_pitch(p.cld);
  T* sk = reinterpret_cast<T*>(smem_raw);              // [kLmKeys][P]
  T* sqh = sk + kLmKeys * P;                           // [16][P] high parts of the queries, then their remainders
  T* sql = sqh + kLmHeads * P;
  float* ss = reinterpret_cast<float*>(sql + kLmHeads * P);          // [16][kLmKeys + 1]
  T* sph = reinterpret_cast<T*>(ss + kLmHeads * (kLmKeys + 1));      // [16][kLmKeys + 8]
  T* spl = sph + kLmHeads * (kLmKeys + 8);
  float* sm_m = reinterpret_cast<float*>(spl + kLmHeads * (kLmKeys + 8));
  float* sm_l = sm_m + kLmHeads;
  float* sm_a = sm_l + kLmHeads;
  const int split = blockIdx.x, r = blockIdx.z, s = r / p.T, t = r % p.T, h0 = (int)blockIdx.y * kLmHeads;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_trigger();
  const int n_keys = min(p.pos[s] + t + 1, p.max_len);
  const int per = ((n_keys + p.splits - 1) / p.splits + kLmKeys - 1) / kLmKeys * kLmKeys;
  const int k_lo = split * per, k_hi = min(n_keys, k_lo + per);
  const int live = min(kLmHeads, p.heads - h0);
  if (k_lo >= k_hi) {                                  // nothing for this split: an empty partial
    for (int i = threadIdx.x; i < live; i += 256) {
      float* dst = p.part + (((long long)r * p.heads + h0 + i) * p.splits + split) * (p.rank + 2);
      dst[0] = -INFINITY; dst[1] = 0.f;
    }
    for (int i = threadIdx.x; i < live * p.rank; i += 256)
      p.part[(((long long)r * p.heads + h0 + i / p.rank) * p.splits + split) * (p.rank + 2) + 2 + i % p.rank] = 0.f;
    return;
  }
  for (int i = threadIdx.x; i < kLmHeads * K; i += 256) {
    const int hh = i / K, c = i % K;
    const float v = hh < live && c < p.cld ? p.q_eff[((long long)r * p.heads + h0 + hh) * p.cld + c] : 0.f;
    const T hi = Cvt<T>::from(v);
    sqh[hh * P + c] = hi;
    sql[hh * P + c] = Cvt<T>::from(v - Cvt<T>::to(hi));
  }
  for (int i = threadIdx.x; i < kLmKeys * (K - p.cld); i += 256) sk[i / (K - p.cld) * P + p.cld + i % (K - p.cld)] = Cvt<T>::from(0.f);
  if (threadIdx.x < kLmHeads) { sm_m[threadIdx.x] = -INFINITY; sm_l[threadIdx.x] = 0.f; }
  const T* cache = reinterpret_cast<const T*>(p.cache) + (long long)s * p.seq_stride;
  float o[NW][4];
#pragma unroll
  for (int j = 0; j < NW; j++) { o[j][0] = 0.f; o[j][1] = 0.f; o[j][2] = 0.f; o[j][3] = 0.f; }
  const int pieces = p.cld / 8;
  for (int k0 = k_lo; k0 < k_hi; k0 += kLmKeys) {
    const int nk = min(kLmKeys, k_hi - k0);
    __syncthreads();
    for (int i = threadIdx.x; i < kLmKeys * pieces; i += 256) {
      const int j = i / pieces, c = i % pieces * 8;
      T* dst = sk + j * P + c;
      if (j < nk) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst)), "l"(cache + (long long)(k0 + j) * p.cld + c));
      else *reinterpret_cast<uint4*>(dst) = make_uint4(0u, 0u, 0u, 0u);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    {
      // scores: 16 heads x 8 keys per warp
      float c4[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t qa = smem_addr(sqh + (lane & 15) * P + (lane >> 4) * 8), la = smem_addr(sql + (lane & 15) * P + (lane >> 4) * 8);
      const uint32_t ka = smem_addr(sk + (warp * 8 + (lane & 7)) * P + (lane >> 3) * 8);
      for (int kk = 0; kk < K; kk += 32) {
        uint32_t b[4], a0[4], a1[4];
        ldsm_x4(b, ka + kk * 2);
        ldsm_x4(a0, qa + kk * 2);
        ldsm_x4(a1, qa + kk * 2 + 32);
        mma_16816<T>(c4, a0[0], a0[1], a0[2], a0[3], b[0], b[1]);
        mma_16816<T>(c4, a1[0], a1[1], a1[2], a1[3], b[2], b[3]);
        ldsm_x4(a0, la + kk * 2);
        ldsm_x4(a1, la + kk * 2 + 32);
        mma_16816<T>(c4, a0[0], a0[1], a0[2], a0[3], b[0], b[1]);
        mma_16816<T>(c4, a1[0], a1[1], a1[2], a1[3], b[2], b[3]);
      }
      const int g = lane >> 2, q = lane & 3, key = warp * 8 + 2 * q;
      ss[g * (kLmKeys + 1) + key] = c4[0]; ss[g * (kLmKeys + 1) + key + 1] = c4[1];
      ss[(g + 8) * (kLmKeys + 1) + key] = c4[2]; ss[(g + 8) * (kLmKeys + 1) + key + 1] = c4[3];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; i++) {
      const int h = warp * 2 + i;
      const float x0 = lane < nk ? ss[h * (kLmKeys + 1) + lane] : -INFINITY, x1 = lane + 32 < nk ? ss[h * (kLmKeys + 1) + lane + 32] : -INFINITY;
      const float m0 = sm_m[h], m1 = fmaxf(m0, warp_max(fmaxf(x0, x1)));
      const float e0 = lane < nk ? expf(x0 - m1) : 0.f, e1 = lane + 32 < nk ? expf(x1 - m1) : 0.f;
      const float sum = warp_sum(e0 + e1);
      const T p0 = Cvt<T>::from(e0), p1 = Cvt<T>::from(e1);
      sph[h * (kLmKeys + 8) + lane] = p0; sph[h * (kLmKeys + 8) + lane + 32] = p1;
      spl[h * (kLmKeys + 8) + lane] = Cvt<T>::from(e0 - Cvt<T>::to(p0)); spl[h * (kLmKeys + 8) + lane + 32] = Cvt<T>::from(e1 - Cvt<T>::to(p1));
      if (lane == 0) {
        const float a = m0 == -INFINITY ? 0.f : expf(m0 - m1);
        sm_a[h] = a; sm_l[h] = sm_l[h] * a + sum; sm_m[h] = m1;
      }
    }
    __syncthreads();
    {
      const int g = lane >> 2;
      const float f0 = sm_a[g], f1 = sm_a[g + 8];
#pragma unroll
      for (int j = 0; j < NW; j++) { o[j][0] *= f0; o[j][1] *= f0; o[j][2] *= f1; o[j][3] *= f1; }
      const uint32_t pa = smem_addr(sph + (lane & 15) * (kLmKeys + 8) + (lane >> 4) * 8), pl = smem_addr(spl + (lane & 15) * (kLmKeys + 8) + (lane >> 4) * 8);
#pragma unroll
      for (int kk = 0; kk < kLmKeys; kk += 32) {
        uint32_t h0a[4], h1a[4], l0a[4], l1a[4];
        ldsm_x4(h0a, pa + kk * 2); ldsm_x4(h1a, pa + kk * 2 + 32);
        ldsm_x4(l0a, pl + kk * 2); ldsm_x4(l1a, pl + kk * 2 + 32);
#pragma unroll
        for (int j = 0; j < NW; j++) {
          const int c = (j * 8 + warp) * 8;
          if (c >= p.rank) break;
          uint32_t b[4];                               // keys kk .. kk + 31 of eight latent columns
          ldsm_x4_t(b, smem_addr(sk + (kk + lane) * P + c));
          mma_16816<T>(o[j], h0a[0], h0a[1], h0a[2], h0a[3], b[0], b[1]);
          mma_16816<T>(o[j], h1a[0], h1a[1], h1a[2], h1a[3], b[2], b[3]);
          mma_16816<T>(o[j], l0a[0], l0a[1], l0a[2], l0a[3], b[0], b[1]);
          mma_16816<T>(o[j], l1a[0], l1a[1], l1a[2], l1a[3], b[2], b[3]);
        }
      }
    }
  }
  const int g = lane >> 2, q = lane & 3;
#pragma unroll
  for (int i = 0; i < 2; i++) {
    const int h = g + 8 * i;
    if (h >= live) continue;
    float* dst = p.part + (((long long)r * p.heads + h0 + h) * p.splits + split) * (p.rank + 2);
    if (warp == 0 && q == 0) { dst[0] = sm_m[h]; dst[1] = sm_l[h]; }
#pragma unroll
    for (int j = 0; j < NW; j++) {
      const int c = (j * 8 + warp) * 8 + 2 * q;
      if (c < p.rank) dst[2 + c] = o[j][2 * i];
      if (c + 1 < p.rank) dst[2 + c + 1] = o[j][2 * i + 1];
    }
  }
}

// merge: the splits of one head combined, then the head's slice of W_uv.
template <typename T>
__global__ void __launch_bounds__(256) latent_decode_merge_kernel(const LaParams p) {
  extern __shared__ __align__(16) float so[];            // [rank]
  __shared__ float s_w[128];
  const int h = blockIdx.x, r = blockIdx.y;
  pdl_wait();
  pdl_trigger();
  const float* part = p.part + ((long long)r * p.heads + h) * p.splits * (p.rank + 2);
  if (threadIdx.x < 32) {
    float m = -INFINITY;
    for (int i = threadIdx.x; i < p.splits; i += 32) m = fmaxf(m, part[(long long)i * (p.rank + 2)]);
    m = warp_max(m);
    float l = 0.f;
    for (int i = threadIdx.x; i < p.splits; i += 32) {
      const float mi = part[(long long)i * (p.rank + 2)];
      const float w = mi == -INFINITY ? 0.f : expf(mi - m);
      s_w[i] = w;
      l += w * part[(long long)i * (p.rank + 2) + 1];
    }
    l = warp_sum(l);
    __syncwarp();
    for (int i = threadIdx.x; i < p.splits; i += 32) s_w[i] /= l;
  }
  __syncthreads();
  for (int c = threadIdx.x; c < p.coff; c += 256) {
    float a = 0.f;
    if (c < p.rank)
#pragma unroll 8
      for (int i = 0; i < p.splits; i++) a = fmaf(s_w[i], part[(long long)i * (p.rank + 2) + 2 + c], a);
    so[c] = a;
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* uv = reinterpret_cast<const T*>(p.uv) + (long long)h * p.vdim * p.w_ld;
  T* y = reinterpret_cast<T*>(p.y) + (long long)r * p.y_ld + (long long)h * p.vdim;
  constexpr int N = Pack<T>::N, R = 4;                   // R rows of W_uv per warp and pass, 16-byte pieces
  const int nv = p.coff / N;
  for (int e0 = warp * R; e0 < p.vdim; e0 += 8 * R) {
    float a[R];
#pragma unroll
    for (int r = 0; r < R; r++) a[r] = 0.f;
    for (int c = lane; c < nv; c += 32) {
      Pack<T> w[R];
#pragma unroll
      for (int r = 0; r < R; r++) w[r] = ld16(uv + (long long)min(e0 + r, p.vdim - 1) * p.w_ld + c * N);
#pragma unroll
      for (int q = 0; q < N; q++) {
        const float x = so[c * N + q];
#pragma unroll
        for (int r = 0; r < R; r++) a[r] = fmaf(x, Cvt<T>::to(w[r].v[q]), a[r]);
      }
    }
#pragma unroll
    for (int r = 0; r < R; r++) {
      a[r] = warp_sum(a[r]);
      if (lane == 0 && e0 + r < p.vdim) y[e0 + r] = Cvt<T>::from(a[r]);
    }
  }
}

static int la_splits(int rows, int heads, int max_len) {
  const int groups = rows * ((heads + kLdHeads - 1) / kLdHeads);
  int want = (2 * 148 + groups - 1) / groups, cap = (max_len + 63) / 64;
  if (want > cap) want = cap;
  return want < 1 ? 1 : (want > 128 ? 128 : want);
}
size_t latent_decode_work_bytes(int rows, int heads, int kv_rank, int rot_dim, int max_len) {
  int worst = 0;                                          // fewer rows may use more splits each
  for (int r = 1; r <= rows; r++) { const int v = r * la_splits(r, heads, max_len); if (v > worst) worst = v; }
  return ((size_t)rows * heads * latent_cache_ld(kv_rank, rot_dim) + 64 + (size_t)worst * heads * (kv_rank + 2)) * sizeof(float) + 512;
}

template <typename T, int NR>
static cudaError_t launch_ld(cudaStream_t s, const LaParams& p, dim3 grid, size_t smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_attend_kernel<T, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  return launch_pdl(latent_decode_attend_kernel<T, NR>, grid, dim3(256), smem, s, p);
}
template <typename T, int NW>
static cudaError_t launch_lm(cudaStream_t s, const LaParams& p, dim3 grid, size_t smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_attend_mma_kernel<T, NW>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  return launch_pdl(latent_decode_attend_mma_kernel<T, NW>, grid, dim3(256), smem, s, p);
}
template <typename T>
static cudaError_t latent_decode_t(cudaStream_t s, const LaParams& p) {
  const int rows = p.n_seq * p.T;
  const size_t psmem = ((size_t)p.dim + 256 * Pack<T>::N) * sizeof(float);
  cudaError_t e = launch_pdl(latent_decode_prepare_kernel<T>, dim3((unsigned)(p.heads + 1), (unsigned)rows), dim3(256), psmem, s, p);
  if (e != cudaSuccess) return e;
  bool done = false;
  if constexpr (sizeof(T) == 2) {
    const size_t smem = lm_smem(p.cld);
    if (smem <= 220 * 1024) {
      const dim3 grid((unsigned)p.splits, (unsigned)((p.heads + kLmHeads - 1) / kLmHeads), (unsigned)rows);
      e = p.rank <= 128 ? launch_lm<T, 2>(s, p, grid, smem) : p.rank <= 256 ? launch_lm<T, 4>(s, p, grid, smem) : p.rank <= 512 ? launch_lm<T, 8>(s, p, grid, smem)
                                                                                                                                : launch_lm<T, 16>(s, p, grid, smem);
      done = true;
    }
  }
  if (!done) {
    const size_t smem = (size_t)kLdHeads * p.cld * sizeof(float) + (size_t)kLdKeys * (p.cld + 2) * sizeof(T);
    const dim3 grid((unsigned)p.splits, (unsigned)((p.heads + kLdHeads - 1) / kLdHeads), (unsigned)rows);
    if (p.rank <= 64) e = launch_ld<T, 2>(s, p, grid, smem);
    else if (p.rank <= 128) e = launch_ld<T, 4>(s, p, grid, smem);
    else if (p.rank <= 256) e = launch_ld<T, 8>(s, p, grid, smem);
    else if (p.rank <= 512) e = launch_ld<T, 16>(s, p, grid, smem);
    else e = launch_ld<T, 32>(s, p, grid, smem);
  }
  if (e != cudaSuccess) return e;
  return launch_pdl(latent_decode_merge_kernel<T>, dim3((unsigned)p.heads, (unsigned)rows), dim3(256), (size_t)p.coff * sizeof(float), s, p);
}

Status latent_decode(cudaStream_t s, const LatentDesc& d, void* work) {
  LaParams p;
  AG_RETURN_IF_ERROR(la_params(d, &p));
  if (!work || !d.w_uk || !d.w_uv || !d.y) return Status::invalid("latent decode: missing operand");
  if (d.n_seq * d.T > 65535 || d.kv_rank > 1024) return Status::unsupported("latent decode: latent rank above 1024");
  const int rows = d.n_seq * d.T;
  p.splits = la_splits(rows, d.heads, d.max_len);
  p.q_eff = static_cast<float*>(work);
  p.part = p.q_eff + ((size_t)rows * d.heads * p.cld + 63) / 64 * 64;
  cudaError_t e = cudaSuccess;
  AG_DISPATCH_FLOAT(d.dtype, T, (e = latent_decode_t<T>(s, p)));
  return cuda_status(e, "latent decode");
}

}}  // namespace ag::k
