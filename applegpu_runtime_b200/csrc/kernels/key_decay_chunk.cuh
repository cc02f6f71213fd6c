// Matrix states with one decay per key channel, prompt portions in chunks of 32 tokens (16-bit storage).
//
// With A_i = a_1 .. a_i the decay of a channel from the chunk's start through token i and S_0 the state in front of the chunk,
//     u_i = beta_i (v_i - (A_i k_i) S_0 - sum_{j<i} K_ij u_j),  K_ij = k_i (A_i / A_j) k_j      (delta rule; otherwise u = v)
//     o_i = (A_i q_i) S_0 + sum_{j<=i} Q_ij u_j,                Q_ij = q_i (A_i / A_j) k_j
//     S   = A_32 S_0 + sum_j (A_32 / A_j k_j) u_j^T.
// (I + beta K) u = beta v - beta (A k) S_0 is solved for both right-hand sides ahead of the state, u = U - W S_0:
//   prepare  every chunk on its own: convolutions, unit norms, decays, Q and K, U and W by forward substitution
//   scan     the chunks of a head one after the other; a warp owns 16 value columns of S as accumulator fragments, so that S,
//            u and the state's update chain from one product to the next without leaving registers
//   finish   the head's norm, its weight and the gate
// No decay is ever inverted: quotients A_i / A_j are products of the decays between j and i. Inside a block of 8 tokens they are
// multiplied up term by term in float32; between blocks they split at block borders into factors of at most one, and the sums
// over channels become small products. Values that the recurrence wants in float32 enter products as the sum of two 16-bit
// numbers, high part and remainder (three products of four), which leaves an error near 2^-17.
#pragma once
#include "key_decay.cuh"
#include "mma_sync.cuh"
#include "sm100.cuh"
#include "tc_math.cuh"
#include <algorithm>

namespace ag { namespace k {

using sm100::mbar_arrive;
using sm100::mbar_expect_tx;
using sm100::mbar_wait;

constexpr int kKdThreads = 256, kKdBlock = 8, kKdBlocks = kKdChunk / kKdBlock;
constexpr int kKdAPitch = kKdChunk + 8;

// What prepare hands to scan for one chunk of one head: planes of [32][dp + 8] (high part, remainder) of A q, then (delta) -W, then
// A_32 / A k, planes of [32][40] of Q, the chunk's decay [dp] in float32.
template <typename T>
struct KdOps {
  T* qg; T* w; T* kg; T* a; float* decay; int plane;
  __device__ KdOps(uint8_t* base, int dp, bool delta) {
    plane = kKdChunk * (dp + 8);
    qg = reinterpret_cast<T*>(base);
    w = qg + 2 * plane;
    kg = w + (delta ? 2 * plane : 0);
    a = kg + 2 * plane;
    decay = reinterpret_cast<float*>(a + 2 * kKdChunk * kKdAPitch);
  }
};

template <typename T>
__device__ __forceinline__ void kd_split(float x, T& hi, T& lo) { hi = Cvt<T>::from(x); lo = Cvt<T>::from(x - Cvt<T>::to(hi)); }
template <typename T>
__device__ __forceinline__ void kd_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack2_t<T>(x, y);
  const T* v = reinterpret_cast<const T*>(&hi);
  lo = pack2_t<T>(x - Cvt<T>::to(v[0]), y - Cvt<T>::to(v[1]));
}

template <typename T, int DP, bool DELTA>
__global__ void __launch_bounds__(kKdThreads) key_decay_prepare_kernel(const KdParams p) {
  constexpr int P = DP + 4, NC = DP / 32;
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                        // [32][P]: q, later q times the decays from its block's start
  float* sk = sq + kKdChunk * P;         // [32][P]: k, later likewise
  float* sa = sk + kKdChunk * P;         // [32][P]: decays, later k times the decays to its block's end
  float* sb = sa + kKdChunk * P;         // [4][DP] decays of whole blocks
  float* sQ = sb + kKdBlocks * DP;       // [32][36]
  float* sK = sQ + kKdChunk * 36;        // [32][36], times beta
  float* s_beta = sK + kKdChunk * 36;    // [32]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c = blockIdx.x, h = blockIdx.y, s = blockIdx.z, qh = h / p.group, D = p.dim, E = p.vdim;
  const int t0 = c * kKdChunk, nt = min(kKdChunk, p.T - t0);
  const long long chunk = ((long long)s * p.heads + h) * p.chunks + c;
  pdl_wait();
  pdl_trigger();
  const int pos = p.pos[s];
  const T* base = reinterpret_cast<const T*>(p.proj) + (long long)s * p.T * p.ld;
  const T* ring = p.ring_of<T>(s);
  KdOps<T> ops(p.ops + chunk * p.ops_bytes, DP, DELTA);
  for (int i = tid; i < kKdChunk * DP; i += kKdThreads) {
    const int t = i / DP, d = i % DP;
    float q = 0.f, k = 0.f, a = 1.f;
    if (t < nt && d < D) {
      const int ch = qh * D + d;
      q = kd_input<T>(p, base, ring, pos, t0 + t, p.q_off + ch, ch);
      k = kd_input<T>(p, base, ring, pos, t0 + t, p.k_off + ch, p.qk_heads * D + ch);
      a = kd_decay(p, h, p.z[((long long)s * p.T + t0 + t) * p.heads * D + h * D + d] + p.bias[h * D + d]);
      if (!p.unit) q *= p.q_scale;
    }
    sq[t * P + d] = q; sk[t * P + d] = k; sa[t * P + d] = a;
  }
  for (int i = tid; i < kKdChunk * 36; i += kKdThreads) { sQ[i] = 0.f; sK[i] = 0.f; }
  if (tid < kKdChunk) s_beta[tid] = DELTA && tid < nt ? sigmoid_f(p.beta[((long long)s * p.T + t0 + tid) * p.beta_ld + h]) : 0.f;
  __syncthreads();
  if (p.unit) {
    for (int t = warp; t < kKdChunk; t += kKdThreads / 32) {
      float qq = 0.f, kk = 0.f;
      for (int d = lane; d < DP; d += 32) { const float a = sq[t * P + d], b = sk[t * P + d]; qq = fmaf(a, a, qq); kk = fmaf(b, b, kk); }
      const float fq = p.q_scale / sqrtf(warp_sum(qq) + 1e-6f), fk = 1.0f / sqrtf(warp_sum(kk) + 1e-6f);
      for (int d = lane; d < DP; d += 32) { sq[t * P + d] *= fq; sk[t * P + d] *= fk; }
    }
    __syncthreads();
  }
  {
    // pairs inside a block: eight lanes per key token j, which carry its decayed key from one query token to the next
    const int j = tid >> 3, sl = tid & 7, last = j / kKdBlock * kKdBlock + kKdBlock - 1;
    float4 kk[NC];
#pragma unroll
    for (int n = 0; n < NC; n++) kk[n] = *reinterpret_cast<const float4*>(sk + j * P + (sl + 8 * n) * 4);
    for (int i = j & ~3; i <= last; i++) {               // the four keys of a warp walk the same rows
      float s1 = 0.f, s2 = 0.f;
#pragma unroll
      for (int n = 0; n < NC; n++) {
        const int at = i * P + (sl + 8 * n) * 4;
        if (i > j) {
          const float4 a = *reinterpret_cast<const float4*>(sa + at);
          kk[n].x *= a.x; kk[n].y *= a.y; kk[n].z *= a.z; kk[n].w *= a.w;
        }
        const float4 q = *reinterpret_cast<const float4*>(sq + at);
        s1 = fmaf(q.x, kk[n].x, fmaf(q.y, kk[n].y, fmaf(q.z, kk[n].z, fmaf(q.w, kk[n].w, s1))));
        if constexpr (DELTA) {
          const float4 k = *reinterpret_cast<const float4*>(sk + at);
          s2 = fmaf(k.x, kk[n].x, fmaf(k.y, kk[n].y, fmaf(k.z, kk[n].z, fmaf(k.w, kk[n].w, s2))));
        }
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) {
        s1 += __shfl_xor_sync(0xffffffffu, s1, o);
        if constexpr (DELTA) s2 += __shfl_xor_sync(0xffffffffu, s2, o);
      }
      if (sl == 0 && i >= j) {
        sQ[i * 36 + j] = s1;
        if (DELTA && i > j) sK[i * 36 + j] = s2 * s_beta[i];
      }
    }
  }
  __syncthreads();
  float w[kKdChunk];                     // this thread's channel of A k, the right-hand side of W
  if (tid < DP) {
    const int d = tid;
    float kk[kKdChunk], pre = 1.f, loc = 1.f;
#pragma unroll
    for (int i = 0; i < kKdChunk; i++) {
      const float a = sa[i * P + d], q = sq[i * P + d];
      kk[i] = sk[i * P + d];
      if (i % kKdBlock == 0) loc = 1.f;
      pre *= a; loc *= a;
      T hi, lo;
      kd_split<T>(q * pre, hi, lo);
      ops.qg[i * (DP + 8) + d] = hi; ops.qg[ops.plane + i * (DP + 8) + d] = lo;
      w[i] = kk[i] * pre;
      sq[i * P + d] = q * loc; sk[i * P + d] = kk[i] * loc;
      if (i % kKdBlock == kKdBlock - 1) sb[i / kKdBlock * DP + d] = loc;
    }
    float suf = 1.f;
    loc = 1.f;
#pragma unroll
    for (int i = kKdChunk - 1; i >= 0; i--) {
      if (i % kKdBlock == kKdBlock - 1) loc = 1.f;
      const float a = sa[i * P + d];
      T hi, lo;
      kd_split<T>(kk[i] * suf, hi, lo);
      ops.kg[i * (DP + 8) + d] = hi; ops.kg[ops.plane + i * (DP + 8) + d] = lo;
      sa[i * P + d] = kk[i] * loc;
      suf *= a; loc *= a;
    }
    ops.decay[d] = suf;
  }
  __syncthreads();
  if (warp < 6) {
    // pairs of different blocks, queries of block b with keys of block a: rows 0 .. 7 of the product are q, rows 8 .. 15 k
    const int b = warp < 1 ? 1 : warp < 3 ? 2 : 3, a = warp - b * (b - 1) / 2, g = lane >> 2, q = lane & 3;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    const float* rq = sq + (b * kKdBlock + g) * P + 2 * q;
    const float* rk = sk + (b * kKdBlock + g) * P + 2 * q;
    const float* rj = sa + (a * kKdBlock + g) * P + 2 * q;
#pragma unroll 2
    for (int k0 = 0; k0 < DP; k0 += 16) {
      uint32_t ah[4], al[4], bh[2], bl[2];
#pragma unroll
      for (int x = 0; x < 2; x++) {
        const int at = k0 + 8 * x;
        const float2 fq = *reinterpret_cast<const float2*>(rq + at);
        kd_split2<T>(fq.x, fq.y, ah[2 * x], al[2 * x]);
        if constexpr (DELTA) {
          const float2 fk = *reinterpret_cast<const float2*>(rk + at);
          kd_split2<T>(fk.x, fk.y, ah[2 * x + 1], al[2 * x + 1]);
        } else { ah[2 * x + 1] = 0u; al[2 * x + 1] = 0u; }
        float2 fj = *reinterpret_cast<const float2*>(rj + at);
        for (int m = a + 1; m < b; m++) { const float2 fb = *reinterpret_cast<const float2*>(sb + m * DP + at + 2 * q); fj.x *= fb.x; fj.y *= fb.y; }
        kd_split2<T>(fj.x, fj.y, bh[x], bl[x]);
      }
      mma_16816<T>(acc, ah[0], ah[1], ah[2], ah[3], bh[0], bh[1]);
      mma_16816<T>(acc, al[0], al[1], al[2], al[3], bh[0], bh[1]);
      mma_16816<T>(acc, ah[0], ah[1], ah[2], ah[3], bl[0], bl[1]);
    }
    const int i = b * kKdBlock + g, j = a * kKdBlock + 2 * q;
    sQ[i * 36 + j] = acc[0]; sQ[i * 36 + j + 1] = acc[1];
    if constexpr (DELTA) { sK[i * 36 + j] = acc[2] * s_beta[i]; sK[i * 36 + j + 1] = acc[3] * s_beta[i]; }
  }
  __syncthreads();
  for (int i = tid; i < kKdChunk * kKdAPitch; i += kKdThreads) {
    const int r = i / kKdAPitch, j = i % kKdAPitch;
    T hi, lo;
    kd_split<T>(j < kKdChunk ? sQ[r * 36 + j] : 0.f, hi, lo);
    ops.a[i] = hi; ops.a[kKdChunk * kKdAPitch + i] = lo;
  }
  // forward substitution, a thread per column: W first, then the value columns
  auto solve = [&](float (&x)[kKdChunk]) {
#pragma unroll
    for (int i = 0; i < kKdChunk; i++) {
      float v = x[i] * s_beta[i];
#pragma unroll
      for (int j = 0; j < i; j += 4) {
        const float4 f = *reinterpret_cast<const float4*>(sK + i * 36 + j);      // zero from the diagonal on
        v = fmaf(-f.x, x[j], v);
        if (j + 1 < i) v = fmaf(-f.y, x[j + 1], v);
        if (j + 2 < i) v = fmaf(-f.z, x[j + 2], v);
        if (j + 3 < i) v = fmaf(-f.w, x[j + 3], v);
      }
      x[i] = v;
    }
  };
  if (DELTA && tid < DP) {
    solve(w);
#pragma unroll
    for (int i = 0; i < kKdChunk; i++) {
      T hi, lo;
      kd_split<T>(-w[i], hi, lo);
      ops.w[i * (DP + 8) + tid] = hi; ops.w[ops.plane + i * (DP + 8) + tid] = lo;
    }
  }
  const int first = DELTA ? DP : 0;
  for (int e = tid < first ? tid + kKdThreads - first : tid - first; e < E; e += kKdThreads) {
    const int ch = h * E + e;
#pragma unroll
    for (int i = 0; i < kKdChunk; i++) w[i] = i < nt ? kd_input<T>(p, base, ring, pos, t0 + i, p.v_off + ch, 2 * p.qk_heads * D + ch) : 0.f;
    if constexpr (DELTA) solve(w);
    float4* u = reinterpret_cast<float4*>(p.u + (chunk * E + e) * kKdChunk);
#pragma unroll
    for (int i = 0; i < kKdChunk; i += 4) u[i / 4] = make_float4(w[i], w[i + 1], w[i + 2], w[i + 3]);
  }
}

// ── scan ────────────────────────────────────────────────────────────────────
// Fragments of the transposed problem: accumulators hold S^T [16 value columns, DP], u^T and o^T [16, 32 tokens]; a pair of
// neighbouring accumulator tiles is one A operand of the next product. The chunks' operands arrive in two stages by bulk copies,
// issued by one lane when every warp is done with the stage.
__device__ __forceinline__ void kd_bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(sm100::smem_u32(dst)), "l"(src), "r"(bytes), "r"(sm100::smem_u32(bar)) : "memory");
}
template <typename T>
__device__ __forceinline__ void kd_frag(const float (&x)[4], const float (&y)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
  kd_split2<T>(x[0], x[1], hi[0], lo[0]);
  kd_split2<T>(x[2], x[3], hi[1], lo[1]);
  kd_split2<T>(y[0], y[1], hi[2], lo[2]);
  kd_split2<T>(y[2], y[3], hi[3], lo[3]);
}

template <typename T, int DP, bool DELTA>
__global__ void __launch_bounds__(256) key_decay_scan_kernel(const KdParams p, int* status) {
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ uint64_t full[2], empty[2];
  constexpr int P = DP + 8, DT = DP / 8, NT = kKdChunk / 8, plane = kKdChunk * P, aplane = kKdChunk * kKdAPitch;
  const int warps = (int)blockDim.x / 32, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  const int h = blockIdx.y, s = blockIdx.z, E = p.vdim, D = p.dim;
  const long long sh = (long long)s * p.heads + h;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; i++) { sm100::mbar_init(&full[i], 1); sm100::mbar_init(&empty[i], (uint32_t)warps); }
    sm100::mbar_fence_init();
  }
  __syncthreads();
  pdl_wait();
  pdl_trigger();
  auto fetch = [&](int c) {
    mbar_expect_tx(&full[c & 1], (uint32_t)p.ops_bytes);
    kd_bulk_load(smem + (c & 1) * p.ops_bytes, p.ops + (sh * p.chunks + c) * p.ops_bytes, (uint32_t)p.ops_bytes, &full[c & 1]);
  };
  if (threadIdx.x == 0) { fetch(0); if (p.chunks > 1) fetch(1); }
  const int e0 = ((int)blockIdx.x * warps + warp) * 16 + g, e1 = e0 + 8;
  float* S = p.state(s) + (long long)h * D * E;
  float st[DT][4];
#pragma unroll
  for (int n = 0; n < DT; n++)
#pragma unroll
    for (int x = 0; x < 4; x++) { const int d = n * 8 + 2 * q + (x & 1), e = x < 2 ? e0 : e1; st[n][x] = d < D && e < E ? S[(long long)d * E + e] : 0.f; }
  // ldmatrix rows of this lane: a token's row for operands [tokens, channels], 8 x 8 tiles (tokens 0-7, k), (0-7, k + 8), (8-15, k), ..
  const int r_n = (lane & 7) + ((lane >> 4) << 3), c_n = ((lane >> 3) & 1) << 3;      // operand as it lies: rows are the product's columns
  const int r_t = (lane & 7) + (((lane >> 3) & 1) << 3), c_t = (lane >> 4) << 3;      // transposed: rows are the product's inner index
  for (int c = 0; c < p.chunks; c++) {
    float u[NT][4], o[NT][4];
    const float* U = p.u + ((sh * p.chunks + c) * E) * kKdChunk + 2 * q;
#pragma unroll
    for (int n = 0; n < NT; n++) {
      const float2 a = e0 < E ? *reinterpret_cast<const float2*>(U + (long long)e0 * kKdChunk + n * 8) : make_float2(0.f, 0.f);
      const float2 b = e1 < E ? *reinterpret_cast<const float2*>(U + (long long)e1 * kKdChunk + n * 8) : make_float2(0.f, 0.f);
      u[n][0] = a.x; u[n][1] = a.y; u[n][2] = b.x; u[n][3] = b.y;
      o[n][0] = 0.f; o[n][1] = 0.f; o[n][2] = 0.f; o[n][3] = 0.f;
    }
    const int sg = c & 1;
    if (threadIdx.x == 0 && c > 0 && c + 1 < p.chunks && mbar_wait(&empty[sg ^ 1], (uint32_t)(((c - 1) >> 1) & 1), status, 61)) fetch(c + 1);
    __syncwarp();
    if (!__all_sync(0xffffffffu, mbar_wait(&full[sg], (uint32_t)((c >> 1) & 1), status, 62))) return;
    const T* qg = reinterpret_cast<const T*>(smem + sg * p.ops_bytes);
    const T* w = qg + 2 * plane;
    const T* kg = w + (DELTA ? 2 * plane : 0);
    const T* am = kg + 2 * plane;
    const float* decay = reinterpret_cast<const float*>(am + 2 * aplane);
#pragma unroll
    for (int ks = 0; ks < DT / 2; ks++) {
      uint32_t ah[4], al[4];
      kd_frag<T>(st[2 * ks], st[2 * ks + 1], ah, al);
      auto apply = [&](const T* op, float (&acc)[NT][4]) {
#pragma unroll
        for (int n = 0; n < NT; n += 2) {
          uint32_t bh[4], bl[4];
          const uint32_t at = smem_addr(op + (n * 8 + r_n) * P + ks * 16 + c_n);
          ldsm_x4(bh, at);
          ldsm_x4(bl, at + plane * 2);
#pragma unroll
          for (int x = 0; x < 2; x++) {
            mma_16816<T>(acc[n + x], ah[0], ah[1], ah[2], ah[3], bh[2 * x], bh[2 * x + 1]);
            mma_16816<T>(acc[n + x], al[0], al[1], al[2], al[3], bh[2 * x], bh[2 * x + 1]);
            mma_16816<T>(acc[n + x], ah[0], ah[1], ah[2], ah[3], bl[2 * x], bl[2 * x + 1]);
          }
        }
      };
      if constexpr (DELTA) apply(w, u);
      apply(qg, o);
    }
#pragma unroll
    for (int n = 0; n < DT; n++) {
      const float2 f = *reinterpret_cast<const float2*>(decay + n * 8 + 2 * q);
      st[n][0] *= f.x; st[n][1] *= f.y; st[n][2] *= f.x; st[n][3] *= f.y;
    }
#pragma unroll
    for (int ks = 0; ks < NT / 2; ks++) {
      uint32_t uh[4], ul[4];
      kd_frag<T>(u[2 * ks], u[2 * ks + 1], uh, ul);      // without the delta rule and convolutions u is the stored v, without a remainder
#pragma unroll
      for (int n = 0; n < NT; n += 2) {
        if (n + 1 < 2 * ks) continue;                    // tokens before these keys
        uint32_t bh[4], bl[4];
        const uint32_t at = smem_addr(am + (n * 8 + r_n) * kKdAPitch + ks * 16 + c_n);
        ldsm_x4(bh, at);
        ldsm_x4(bl, at + aplane * 2);
#pragma unroll
        for (int x = 0; x < 2; x++) {
          mma_16816<T>(o[n + x], uh[0], uh[1], uh[2], uh[3], bh[2 * x], bh[2 * x + 1]);
          if (DELTA || p.taps) mma_16816<T>(o[n + x], ul[0], ul[1], ul[2], ul[3], bh[2 * x], bh[2 * x + 1]);
          mma_16816<T>(o[n + x], uh[0], uh[1], uh[2], uh[3], bl[2 * x], bl[2 * x + 1]);
        }
      }
#pragma unroll
      for (int n = 0; n < DT; n += 2) {
        uint32_t bh[4], bl[4];
        const uint32_t at = smem_addr(kg + (ks * 16 + r_t) * P + n * 8 + c_t);
        ldsm_x4_t(bh, at);
        ldsm_x4_t(bl, at + plane * 2);
#pragma unroll
        for (int x = 0; x < 2; x++) {
          mma_16816<T>(st[n + x], uh[0], uh[1], uh[2], uh[3], bh[2 * x], bh[2 * x + 1]);
          if (DELTA || p.taps) mma_16816<T>(st[n + x], ul[0], ul[1], ul[2], ul[3], bh[2 * x], bh[2 * x + 1]);
          mma_16816<T>(st[n + x], uh[0], uh[1], uh[2], uh[3], bl[2 * x], bl[2 * x + 1]);
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[sg]);
    const int t0 = c * kKdChunk + 2 * q;
    float* O = p.o + ((long long)s * p.T * p.heads + h) * E;
#pragma unroll
    for (int n = 0; n < NT; n++)
#pragma unroll
      for (int x = 0; x < 4; x++) {
        const int t = t0 + n * 8 + (x & 1), e = x < 2 ? e0 : e1;
        if (t < p.T && e < E) O[(long long)t * p.heads * E + e] = o[n][x];
      }
  }
#pragma unroll
  for (int n = 0; n < DT; n++)
#pragma unroll
    for (int x = 0; x < 4; x++) { const int d = n * 8 + 2 * q + (x & 1), e = x < 2 ? e0 : e1; if (d < D && e < E) S[(long long)d * E + e] = st[n][x]; }
}

// ── finish: norm and gate of one head's outputs, a warp each ────────────────
template <typename T, int VEC>
__global__ void __launch_bounds__(256) key_decay_finish_kernel(const KdParams p) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31, E = p.vdim;
  const long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5), rows = (long long)p.n_seq * p.T;
  if (i >= rows * p.heads) return;
  const long long r = i / p.heads;
  const int h = (int)(i % p.heads);
  const float* o = p.o + i * E;
  const T* gate = p.gate ? reinterpret_cast<const T*>(p.gate) + r * p.gate_ld + (long long)h * E : reinterpret_cast<const T*>(p.proj) + r * p.ld + p.g_off + (long long)h * E;
  T* y = reinterpret_cast<T*>(p.y) + r * p.y_ld + (long long)h * E;
  float sq = 0.f;
  for (int e = lane * VEC; e < E; e += 32 * VEC) {
    if constexpr (VEC == 4) { const float4 v = *reinterpret_cast<const float4*>(o + e); sq = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, sq)))); }
    else sq = fmaf(o[e], o[e], sq);
  }
  const float rs = 1.0f / sqrtf(warp_sum(sq) / (float)E + p.eps);
  for (int e = lane * VEC; e < E; e += 32 * VEC) {
    if constexpr (VEC == 4) {
      const float4 v = *reinterpret_cast<const float4*>(o + e), w = *reinterpret_cast<const float4*>(p.norm + e);
      const uint2 graw = *reinterpret_cast<const uint2*>(gate + e);
      const T* gv = reinterpret_cast<const T*>(&graw);
      uint2 out;
      out.x = pack2_t<T>(v.x * rs * w.x * kd_gate(p, Cvt<T>::to(gv[0])), v.y * rs * w.y * kd_gate(p, Cvt<T>::to(gv[1])));
      out.y = pack2_t<T>(v.z * rs * w.z * kd_gate(p, Cvt<T>::to(gv[2])), v.w * rs * w.w * kd_gate(p, Cvt<T>::to(gv[3])));
      *reinterpret_cast<uint2*>(y + e) = out;
    } else y[e] = Cvt<T>::from(o[e] * rs * p.norm[e] * kd_gate(p, Cvt<T>::to(gate[e])));
  }
}

// ── host ────────────────────────────────────────────────────────────────────
template <typename T, int DP, bool DELTA>
static cudaError_t launch_kd(cudaStream_t s, const KdParams& p, int warps) {
  constexpr size_t prep = ((size_t)3 * kKdChunk * (DP + 4) + kKdBlocks * DP + 2 * kKdChunk * 36 + kKdChunk) * sizeof(float);
  const size_t scan = 2 * (size_t)p.ops_bytes;
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(key_decay_prepare_kernel<T, DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)prep);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(key_decay_scan_kernel<T, DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  cudaError_t e = launch_pdl(key_decay_prepare_kernel<T, DP, DELTA>, dim3((unsigned)p.chunks, (unsigned)p.heads, (unsigned)p.n_seq), dim3(kKdThreads), prep, s, p);
  if (e != cudaSuccess) return e;
  const unsigned slices = (unsigned)((p.vdim + 16 * warps - 1) / (16 * warps));
  return launch_pdl(key_decay_scan_kernel<T, DP, DELTA>, dim3(slices, (unsigned)p.heads, (unsigned)p.n_seq), dim3((unsigned)warps * 32), scan, s, p, matmul_status_word());
}
template <typename T, bool DELTA>
static cudaError_t launch_kd_dp(cudaStream_t s, const KdParams& p, int warps) {
  switch (p.dp) {
    case 32: return launch_kd<T, 32, DELTA>(s, p, warps);
    case 64: return launch_kd<T, 64, DELTA>(s, p, warps);
    case 96: return launch_kd<T, 96, DELTA>(s, p, warps);
    case 128: return launch_kd<T, 128, DELTA>(s, p, warps);
    case 192: return launch_kd<T, 192, DELTA>(s, p, warps);
    default: return launch_kd<T, 256, DELTA>(s, p, warps);
  }
}
template <typename T>
static Status launch_chunked(cudaStream_t s, const KdParams& p) {
  // value columns per CTA: up to 128, fewer where that leaves SMs without work
  int warps = std::min(8, (p.vdim + 15) / 16);
  while (warps > 2 && (long long)p.n_seq * p.heads * ((p.vdim + 16 * warps - 1) / (16 * warps)) < sm_count()) warps = (warps + 1) / 2;
  cudaError_t e = p.delta ? launch_kd_dp<T, true>(s, p, warps) : launch_kd_dp<T, false>(s, p, warps);
  if (e != cudaSuccess) return cuda_status(e, "key decay (chunked)");
  const unsigned blocks = (unsigned)(((long long)p.n_seq * p.T * p.heads + 7) / 8);
  const bool vec = p.vdim % 4 == 0 && p.y_ld % 4 == 0 && aligned16(p.y) && aligned16(p.norm) && (p.gate ? p.gate_ld % 4 == 0 : p.ld % 4 == 0 && p.g_off % 4 == 0 && aligned16(p.proj));
  e = vec ? launch_pdl(key_decay_finish_kernel<T, 4>, dim3(blocks), dim3(256), 0, s, p) : launch_pdl(key_decay_finish_kernel<T, 1>, dim3(blocks), dim3(256), 0, s, p);
  return cuda_status(e, "key decay (chunked)");
}

}}  // namespace ag::k
