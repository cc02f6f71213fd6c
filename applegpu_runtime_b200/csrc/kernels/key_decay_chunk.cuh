// Matrix states with one decay per key channel, prompt portions in chunks of 32 tokens (16-bit storage).
//
// With A_i = a_1 .. a_i the decay of a channel from the chunk's start through token i and S_0 the state in front of the chunk,
//     u_i = beta_i (v_i - (A_i k_i) S_0 - sum_{j<i} K_ij u_j),  K_ij = k_i (A_i / A_j) k_j      (delta rule; otherwise u = v)
//     o_i = (A_i q_i) S_0 + sum_{j<=i} Q_ij u_j,                Q_ij = q_i (A_i / A_j) k_j
//     S   = A_32 S_0 + sum_j (A_32 / A_j k_j) u_j^T,
// so that u = T (beta v - beta (A k) S_0) with T = (I + beta K)^-1, unit lower triangular.
//   prepare  every chunk on its own: convolutions, unit norms, decays, Q and T (by forward substitution), the scaled rows of q and k
//   scan     the chunks of a head one after the other, the transposed problem on tcgen05: S^T [value columns, channels], u^T and
//            o^T are accumulators in tensor memory, S^T and u^T (split) A operands there; up to 128 channels and 128 value columns per
//            CTA. Where that is all of a head, its norm, norm weight and gate follow, one chunk behind, in warps of their own.
//            Wider keys take a warp-level form: a warp owns 16 value columns, its accumulator fragments chain in registers; the
//            prepare kernel solves for both right-hand sides there, u = U - W S_0
//   finish   norm and gate of wider heads
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
#include <type_traits>

namespace ag { namespace k {

using sm100::mbar_arrive;
using sm100::mbar_expect_tx;
using sm100::mbar_wait;

constexpr int kKdThreads = 256, kKdBlock = 8, kKdBlocks = kKdChunk / kKdBlock;

template <typename T>
__device__ __forceinline__ void kd_split(float x, T& hi, T& lo) { hi = Cvt<T>::from(x); lo = Cvt<T>::from(x - Cvt<T>::to(hi)); }
// PACKED: the remainders of the pair in one operation (which form the register allocation favours differs by kernel)
template <typename T, bool PACKED = false>
__device__ __forceinline__ void kd_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack2_t<T>(x, y);
  const T* v = reinterpret_cast<const T*>(&hi);
  float a = x - Cvt<T>::to(v[0]), b = y - Cvt<T>::to(v[1]);
  if constexpr (PACKED) unpack_f32x2(fma_f32x2(pack_f32x2(Cvt<T>::to(v[0]), Cvt<T>::to(v[1])), pack_f32x2(-1.0f, -1.0f), pack_f32x2(x, y)), a, b);
  lo = pack2_t<T>(a, b);
}

__device__ __forceinline__ float kd_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
constexpr float kKdLog2e = 1.4426950408889634f;
// log(1 + e) for 0 <= e <= 1 as 2 artanh(e / (2 + e)), the series of which converges within 1e-7 of the value there
__device__ __forceinline__ float kd_log1p_unit(float e) {
  const float s = e * kd_rcp(2.0f + e), t = s * s;
  float r = fmaf(t, 1.0f / 13.0f, 1.0f / 11.0f);
  r = fmaf(t, r, 1.0f / 9.0f);
  r = fmaf(t, r, 1.0f / 7.0f);
  r = fmaf(t, r, 1.0f / 5.0f);
  r = fmaf(t, r, 1.0f / 3.0f);
  return 2.0f * fmaf(s * t, r, s);
}
__device__ __forceinline__ float kd_softplus_fast(float x) { return fmaxf(x, 0.f) + kd_log1p_unit(ex2_approx(-kKdLog2e * fabsf(x))); }
// exp(f softplus(x)): a decay from its input z, x = z and f = -rate or x = -z and f = -1 / tau; f comes in log2 units
__device__ __forceinline__ float kd_decay_fast(float f_log2, float x) { return ex2_approx(f_log2 * kd_softplus_fast(x)); }
__device__ __forceinline__ float kd_sigmoid_fast(float x) { return kd_rcp(1.0f + ex2_approx(-kKdLog2e * x)); }
__device__ __forceinline__ float kd_gate_fast(const KdParams& p, float x) { const float s = kd_sigmoid_fast(x); return p.gate_silu ? x * s : s; }
__device__ __forceinline__ float kd_silu_fast(float x) { return x * kd_sigmoid_fast(x); }

// Convolutions of up to kKdTaps taps slide over their raw inputs; longer ones read them tap by tap.
constexpr int kKdTaps = 4;
// The taps of channel ch, zeros in front
__device__ __forceinline__ void kd_taps(const KdParams& p, int ch, float (&w)[kKdTaps]) {
#pragma unroll
  for (int j = 0; j < kKdTaps; j++) { const int at = j - (kKdTaps - p.taps); w[j] = at >= 0 ? __ldg(p.conv + (long long)ch * p.taps + at) : 0.f; }
}
// A 16-bit element in a register of its own: an array of these is not packed in pairs, which would wait for the loads
template <typename T> __device__ __forceinline__ uint32_t kd_bits(const T* at) { return *reinterpret_cast<const uint16_t*>(at); }
template <typename T> __device__ __forceinline__ float kd_value(uint32_t bits) {
  const uint16_t b = (uint16_t)bits;
  return Cvt<T>::to(*reinterpret_cast<const T*>(&b));
}
template <> __device__ __forceinline__ float kd_value<__nv_bfloat16>(uint32_t bits) { return __uint_as_float(bits << 16); }
template <typename T>
__device__ __forceinline__ uint32_t kd_round_bits(float x) { const T v = Cvt<T>::from(x); return kd_bits<T>(&v); }
template <typename T>
__device__ __forceinline__ float2 kd_pair(const T* at) {
  const uint32_t raw = *reinterpret_cast<const uint32_t*>(at);
  const T* v = reinterpret_cast<const T*>(&raw);
  return make_float2(Cvt<T>::to(v[0]), Cvt<T>::to(v[1]));
}

template <typename T, int DP, bool DELTA>
__global__ void __launch_bounds__(kKdThreads, kd_tc(DP) ? 3 : DP <= 192 ? 2 : 1) key_decay_prepare_kernel(const KdParams p) {
  constexpr int P = DP + 4, NC = DP / 32, DH = DP / 2;
  constexpr KdOpsLayout L = kd_ops_layout(DP, DELTA);
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                        // [32][P]: q, later q times the decays from its block's start
  float* sk = sq + kKdChunk * P;         // [32][P]: k, later likewise
  float* sa = sk + kKdChunk * P;         // [32][P]: decays, later k times the decays to its block's end
  float* sb = sa + kKdChunk * P;         // [4][DP] decays of whole blocks
  float* sQ = sb + kKdBlocks * DP;       // [32][36]
  float* sK = sQ + kKdChunk * 36;        // [32][36], times beta
  float* s_beta = sK + kKdChunk * 36;    // [32]
  float* s_one = s_beta + 3 * kKdChunk;  // [DP] ones
  float2* s_f = reinterpret_cast<float2*>(s_beta + kKdChunk);      // [32] what makes q and k unit vectors
  float* s_part = s_one + DP;            // [4][6][16][8] shares of the products between blocks
  float* s_pre = s_part;                 // [4][DP] then the decays of the blocks before one, and behind it
  float* s_suf = s_pre + kKdBlocks * DP;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c = blockIdx.x, h = blockIdx.y, s = blockIdx.z, qh = h / p.group, D = p.dim, E = p.vdim;
  const int t0 = c * kKdChunk, nt = min(kKdChunk, p.T - t0);
  const long long chunk = ((long long)s * p.heads + h) * p.chunks + c;
  pdl_wait();
  pdl_trigger();
  const int pos = p.pos[s];
  const T* base = reinterpret_cast<const T*>(p.proj) + (long long)s * p.T * p.ld;
  const T* ring = p.ring_of<T>(s);
  uint8_t* ops = p.ops + chunk * L.stride;
  // one value column over the chunk, and its u (warp-level scan)
  constexpr bool kSolveValues = !kd_tc(DP);
  auto load_v = [&](int e, float (&w)[kKdChunk]) {
    const int ch = h * E + e, rc = 2 * p.qk_heads * D + ch;
    const T* src = base + (long long)t0 * p.ld + p.v_off + ch;
    if (p.taps > kKdTaps) {
#pragma unroll 1
      for (int i = 0; i < kKdChunk; i++) {
        const float v = i < nt ? kd_input<T>(p, base, ring, pos, t0 + i, p.v_off + ch, rc) : 0.f;
#pragma unroll
        for (int j = 0; j < kKdChunk; j++) if (j == i) w[j] = v;
      }
      return;
    }
    if (nt == kKdChunk) {
#pragma unroll
      for (int i = 0; i < kKdChunk; i++) w[i] = Cvt<T>::to(src[(long long)i * p.ld]);
    } else {
#pragma unroll
      for (int i = 0; i < kKdChunk; i++) w[i] = i < nt ? Cvt<T>::to(src[(long long)i * p.ld]) : 0.f;
    }
    if (p.taps == 0) return;
    float f[kKdTaps], x[kKdTaps - 1];
    kd_taps(p, rc, f);
#pragma unroll
    for (int j = 0; j < kKdTaps - 1; j++) { const int back = kKdTaps - 1 - j; x[j] = back < p.taps ? kd_raw<T>(p, base, ring, pos, t0 - back, p.v_off + ch, rc) : 0.f; }
#pragma unroll
    for (int i = kKdChunk - 1; i >= 0; i--) {            // from the end, so that raw inputs are still there
      float y = f[3] * w[i];
#pragma unroll
      for (int n = 1; n < kKdTaps; n++) y = fmaf(f[3 - n], i >= n ? w[i >= n ? i - n : 0] : x[i >= n ? 0 : kKdTaps - 1 + i - n], y);
      w[i] = i < nt ? kd_silu_fast(y) : 0.f;
    }
  };
  auto store_u = [&](int e, const float (&w)[kKdChunk]) {
    float4* u = reinterpret_cast<float4*>(p.u + (chunk * E + e) * kKdChunk);
#pragma unroll
    for (int i = 0; i < kKdChunk; i += 4) u[i / 4] = make_float4(w[i], w[i + 1], w[i + 2], w[i + 3]);
  };
  float w[kKdChunk];                     // a right-hand side: this thread's channel of A k, or (threads past the channels) a value column
  const int e_own = tid - DP;
  const float sign = p.softplus ? 1.f : -1.f, f_log2 = -kKdLog2e * (p.softplus ? p.rate[h] : p.inv_tau);
  if (D % 2 == 0 && p.taps <= kKdTaps) {
    // two channels at a time; everything is requested before anything is used
    constexpr int R = kKdThreads / DH, NZ = (kKdChunk + R - 1) / R;      // tokens per pass, passes
    const int zd = tid % DH * 2, zt = tid / DH;
    const bool z_mine = tid < R * DH, z_live = z_mine && zd < D;
    const float* zp = p.z + ((long long)s * p.T + t0 + zt) * p.heads * D + h * D + zd;
    const long long z_step = (long long)R * p.heads * D;
    float2 z[NZ];
#pragma unroll
    for (int n = 0; n < NZ; n++, zp += z_step) z[n] = z_live && zt + n * R < nt ? __ldcs(reinterpret_cast<const float2*>(zp)) : make_float2(0.f, 0.f);
    const float b0 = z_live ? __ldg(p.bias + h * D + zd) : 0.f, b1 = z_live ? __ldg(p.bias + h * D + zd + 1) : 0.f;
    if (kSolveValues && DELTA && e_own >= 0 && e_own < E) load_v(e_own, w);
    for (int i = tid; i < kKdBlocks * DH; i += kKdThreads) {
      const int d = i % DH * 2, o = i / DH * kKdBlock, first = t0 + o - (kKdTaps - 1);
      constexpr int N = kKdBlock + kKdTaps - 1;
      const bool inside = d < D && first >= 0 && first + N <= p.T;
#pragma unroll 1
      for (int m = 0; m < 2; m++) {
        float2 x[N];
        const int col = (m ? p.k_off : p.q_off) + qh * D + d, ch = (m ? p.qk_heads * D : 0) + qh * D + d;
        const T* src = base + (long long)first * p.ld + col;
        if (inside) {
#pragma unroll
          for (int j = 0; j < N; j++, src += p.ld) x[j] = kd_pair<T>(src);
        } else {
#pragma unroll
          for (int j = 0; j < N; j++) {
            const int t = first + j;
            x[j] = make_float2(0.f, 0.f);
            if (d >= D || t >= p.T || (t < 0 && -t >= p.taps)) continue;
            x[j] = t >= 0 ? kd_pair<T>(src + (long long)j * p.ld) : make_float2(kd_raw<T>(p, base, ring, pos, t, col, ch), kd_raw<T>(p, base, ring, pos, t, col + 1, ch + 1));
          }
        }
        float* dst = (m ? sk : sq) + o * P + d;
        if (p.taps) {
          float w0[kKdTaps], w1[kKdTaps];
          const int wch = ch - d + min(d, D - 2);
          kd_taps(p, wch, w0);
          kd_taps(p, wch + 1, w1);
#pragma unroll
          for (int j = 0; j < kKdBlock; j++) {
            uint64_t sum = 0ull;
#pragma unroll
            for (int n = 0; n < kKdTaps; n++) sum = fma_f32x2(pack_f32x2(w0[n], w1[n]), pack_f32x2(x[j + n].x, x[j + n].y), sum);
            float2 y;
            unpack_f32x2(sum, y.x, y.y);
            *reinterpret_cast<float2*>(dst + j * P) = make_float2(kd_silu_fast(y.x), kd_silu_fast(y.y));      // channels past D are zero already
          }
          if (o + kKdBlock > nt)                         // tokens past the end are not
            for (int j = max(0, nt - o); j < kKdBlock; j++) *reinterpret_cast<float2*>(dst + j * P) = make_float2(0.f, 0.f);
        } else {
#pragma unroll
          for (int j = 0; j < kKdBlock; j++) *reinterpret_cast<float2*>(dst + j * P) = x[j + kKdTaps - 1];
        }
      }
    }
    if (z_mine) {
#pragma unroll
      for (int n = 0; n < NZ; n++) {
        const int t = zt + n * R;
        if (NZ * R > kKdChunk && t >= kKdChunk) break;
        const bool live = z_live && t < nt;
        const float a0 = kd_decay_fast(f_log2, sign * (z[n].x + b0)), a1 = kd_decay_fast(f_log2, sign * (z[n].y + b1));
        *reinterpret_cast<float2*>(sa + t * P + zd) = make_float2(live ? a0 : 1.f, live ? a1 : 1.f);
      }
    }
  } else {
    for (int i = tid; i < kKdChunk * DP; i += kKdThreads) {
      const int t = i / DP, d = i % DP;
      float q = 0.f, k = 0.f, a = 1.f;
      if (t < nt && d < D) {
        const int ch = qh * D + d;
        q = kd_input<T>(p, base, ring, pos, t0 + t, p.q_off + ch, ch);
        k = kd_input<T>(p, base, ring, pos, t0 + t, p.k_off + ch, p.qk_heads * D + ch);
        a = kd_decay_fast(f_log2, sign * (p.z[((long long)s * p.T + t0 + t) * p.heads * D + h * D + d] + p.bias[h * D + d]));
      }
      sq[t * P + d] = q; sk[t * P + d] = k; sa[t * P + d] = a;
    }
    if (kSolveValues && DELTA && e_own >= 0 && e_own < E) load_v(e_own, w);
  }
  if constexpr (kSolveValues && !DELTA) for (int e = tid; e < E; e += kKdThreads) { load_v(e, w); store_u(e, w); }
  for (int i = tid; i < kKdChunk * 36 / 2; i += kKdThreads) reinterpret_cast<float4*>(sQ)[i] = make_float4(0.f, 0.f, 0.f, 0.f);      // Q and K
  if (tid < DP) s_one[tid] = 1.f;
  if (tid < kKdChunk) s_beta[tid] = DELTA && tid < nt ? sigmoid_f(p.beta[((long long)s * p.T + t0 + tid) * p.beta_ld + h]) : 0.f;
  __syncthreads();
  {
    // pairs inside a block: eight lanes per key token j, which carry its decayed key from one query token to the next (two channels to
    // an operation); before that the lengths of the token's own q and k
    const int j = tid >> 3, sl = tid & 7, last = j / kKdBlock * kKdBlock + kKdBlock - 1;
    uint64_t kk[2 * NC];
    auto row = [&](const float* x, int n) { return *reinterpret_cast<const ulonglong2*>(x + (sl + 8 * n) * 4); };
    uint64_t a1 = 0ull, a2 = 0ull;
#pragma unroll
    for (int n = 0; n < NC; n++) {
      const ulonglong2 k = row(sk + j * P, n), q = row(sq + j * P, n);
      kk[2 * n] = k.x; kk[2 * n + 1] = k.y;
      a1 = fma_f32x2(q.x, q.x, fma_f32x2(q.y, q.y, a1));
      a2 = fma_f32x2(k.x, k.x, fma_f32x2(k.y, k.y, a2));
    }
    auto over_lanes = [&](float v) {
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      return v;
    };
    {
      const float qq = over_lanes(sum_f32x2(a1)), kq = over_lanes(sum_f32x2(a2));
      if (sl == 0) s_f[j] = p.unit ? make_float2(p.q_scale / sqrtf(qq + 1e-6f), 1.0f / sqrtf(kq + 1e-6f)) : make_float2(p.q_scale, 1.f);
    }
    for (int i = j & ~3; i <= last; i++) {               // the four keys of a warp walk the same rows
      const float* fade = i > j ? sa + i * P : s_one;
      a1 = 0ull; a2 = 0ull;
#pragma unroll
      for (int n = 0; n < NC; n++) {
        const ulonglong2 a = row(fade, n), q = row(sq + i * P, n);
        kk[2 * n] = mul_f32x2(kk[2 * n], a.x); kk[2 * n + 1] = mul_f32x2(kk[2 * n + 1], a.y);
        a1 = fma_f32x2(q.x, kk[2 * n], fma_f32x2(q.y, kk[2 * n + 1], a1));
        if constexpr (DELTA) {
          const ulonglong2 k = row(sk + i * P, n);
          a2 = fma_f32x2(k.x, kk[2 * n], fma_f32x2(k.y, kk[2 * n + 1], a2));
        }
      }
      const float s1 = over_lanes(sum_f32x2(a1)), s2 = DELTA ? over_lanes(sum_f32x2(a2)) : 0.f;
      if (sl == 0 && i >= j) {
        sQ[i * 36 + j] = s1;
        if (DELTA && i > j) sK[i * 36 + j] = s2 * s_beta[i];
      }
    }
  }
  __syncthreads();
  {                                      // those pairs with the factors of their rows
    const int i = tid >> 3, j = i / kKdBlock * kKdBlock + (tid & 7);
    const float2 fi = s_f[i];
    const float fk = s_f[j].y;
    sQ[i * 36 + j] *= fi.x * fk;
    if constexpr (DELTA) sK[i * 36 + j] *= fi.y * fk;
  }
  // q, k and the keys of a block with the decays from the block's start or to its end
  for (int i = tid; i < kKdBlocks * DP; i += kKdThreads) {
    const int d = i % DP, b = i / DP;
    float* q = sq + b * kKdBlock * P + d;
    float* k = sk + b * kKdBlock * P + d;
    float* a = sa + b * kKdBlock * P + d;
    float kk[kKdBlock], aa[kKdBlock], f = 1.f;
#pragma unroll
    for (int j = 0; j < kKdBlock; j++) {
      const float2 n = s_f[b * kKdBlock + j];
      aa[j] = a[j * P];
      kk[j] = k[j * P] * n.y;
      f *= aa[j];
      q[j * P] *= n.x * f;
      k[j * P] = kk[j] * f;
    }
    sb[b * DP + d] = f;
    f = 1.f;
#pragma unroll
    for (int j = kKdBlock - 1; j >= 0; j--) { a[j * P] = kk[j] * f; f *= aa[j]; }
  }
  __syncthreads();
  // pairs of different blocks, queries of block b with keys of block a < b: rows 0 .. 7 of a product are q, rows 8 .. 15 k. Four warps
  // take every fourth 16 channels of all six.
  constexpr int kShares = DP / 16 < 4 ? DP / 16 : 4;
  if (warp < kShares) {
    const int g = lane >> 2, q = lane & 3;
    float acc[6][4];
#pragma unroll
    for (int i = 0; i < 6; i++) { acc[i][0] = 0.f; acc[i][1] = 0.f; acc[i][2] = 0.f; acc[i][3] = 0.f; }
#pragma unroll 1
    for (int k0 = warp * 16; k0 < DP; k0 += kShares * 16) {
      uint32_t ah[3][4], al[3][4];
      const int c0 = k0 + 2 * q;
      auto at = [&](const float* x, int r, int c) { return *reinterpret_cast<const float2*>(x + r * P + c); };
#pragma unroll
      for (int b = 1; b < kKdBlocks; b++)
#pragma unroll
        for (int x = 0; x < 2; x++) {
          const float2 fq = at(sq, b * kKdBlock + g, c0 + 8 * x);
          kd_split2<T>(fq.x, fq.y, ah[b - 1][2 * x], al[b - 1][2 * x]);
          ah[b - 1][2 * x + 1] = 0u; al[b - 1][2 * x + 1] = 0u;
          if constexpr (DELTA) {
            const float2 fk = at(sk, b * kKdBlock + g, c0 + 8 * x);
            kd_split2<T>(fk.x, fk.y, ah[b - 1][2 * x + 1], al[b - 1][2 * x + 1]);
          }
        }
#pragma unroll
      for (int a = 0; a < kKdBlocks - 1; a++) {
        float2 f[2] = {at(sa, a * kKdBlock + g, c0), at(sa, a * kKdBlock + g, c0 + 8)};
#pragma unroll
        for (int b = a + 1; b < kKdBlocks; b++) {
          uint32_t bh[2], bl[2];
          float (&cc)[4] = acc[b * (b - 1) / 2 + a];
#pragma unroll
          for (int x = 0; x < 2; x++) {
            if (b > a + 1) { const float2 m = *reinterpret_cast<const float2*>(sb + (b - 1) * DP + c0 + 8 * x); f[x].x *= m.x; f[x].y *= m.y; }
            kd_split2<T>(f[x].x, f[x].y, bh[x], bl[x]);
          }
          mma_16816<T>(cc, ah[b - 1][0], ah[b - 1][1], ah[b - 1][2], ah[b - 1][3], bh[0], bh[1]);
          mma_16816<T>(cc, al[b - 1][0], al[b - 1][1], al[b - 1][2], al[b - 1][3], bh[0], bh[1]);
          mma_16816<T>(cc, ah[b - 1][0], ah[b - 1][1], ah[b - 1][2], ah[b - 1][3], bl[0], bl[1]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 6; i++) {
      float* to = s_part + warp * 768 + i * 128 + g * 8 + 2 * q;
      *reinterpret_cast<float2*>(to) = make_float2(acc[i][0], acc[i][1]);
      *reinterpret_cast<float2*>(to + 64) = make_float2(acc[i][2], acc[i][3]);
    }
  }
  __syncthreads();
#pragma unroll
  for (int n = 0; n < 3; n++) {
    const int i = tid + n * kKdThreads, pair = i >> 7, r = (i >> 3) & 15, j = i & 7;
    float v = 0.f;
#pragma unroll
    for (int m = 0; m < kShares; m++) v += s_part[m * 768 + i];
    const int b = pair < 1 ? 1 : pair < 3 ? 2 : 3, a = pair - b * (b - 1) / 2, row = b * kKdBlock + (r & 7), col = a * kKdBlock + j;
    if (r < 8) sQ[row * 36 + col] = v;
    else if constexpr (DELTA) sK[row * 36 + col] = v * s_beta[row];
  }
  __syncthreads();
  if (tid < DP) {                        // a chunk's decays across blocks
    const float f0 = sb[tid], f1 = sb[DP + tid], f2 = sb[2 * DP + tid], f3 = sb[3 * DP + tid];
    s_pre[tid] = 1.f; s_pre[DP + tid] = f0; s_pre[2 * DP + tid] = f0 * f1; s_pre[3 * DP + tid] = f0 * f1 * f2;
    s_suf[tid] = f1 * f2 * f3; s_suf[DP + tid] = f2 * f3; s_suf[2 * DP + tid] = f3; s_suf[3 * DP + tid] = 1.f;
    reinterpret_cast<float*>(ops + L.decay)[tid] = f0 * f1 * f2 * f3;
  }
  __syncthreads();
  const auto store_q = [&](int i, int j) {               // four entries of Q
    const float4 v = *reinterpret_cast<const float4*>(sQ + i * 36 + j);
    uint2 hi, lo;
    kd_split2<T>(v.x, v.y, hi.x, lo.x);
    kd_split2<T>(v.z, v.w, hi.y, lo.y);
    uint8_t* at = ops + L.q + (kd_tc(DP) ? i * 128 : i * kKdAPitch * 2);
    *reinterpret_cast<uint2*>(at + (kd_tc(DP) ? (j * 2) ^ ((i & 7) << 4) : j * 2)) = hi;
    *reinterpret_cast<uint2*>(at + (kd_tc(DP) ? (64 + j * 2) ^ ((i & 7) << 4) : kKdChunk * kKdAPitch * 2 + j * 2)) = lo;
  };
  // rows of A q, A k and A_32 / A k, eight channels at a time
  const auto store_rows = [&](int first, int threads) {
    for (int i = first; i < kKdChunk * DP / 8; i += threads) {
      const int r = i / (DP / 8), unit = i % (DP / 8), b = r / kKdBlock, d = unit * 8;
      // panels: a row's 16-byte pieces are swapped by its number's low bits
      uint8_t* at = ops + (kd_tc(DP) ? r * 128 + (((unit & 7) ^ (r & 7)) << 4) : r * (DP + 8) * 2 + unit * 16);
      const int panel1 = kd_tc(DP) ? (unit >> 3) * 2 * L.plane1 : 0, panel2 = kd_tc(DP) ? (unit >> 3) * kKdChunk * 128 : 0;
      auto put = [&](uint8_t* to, int to_lo, const float* x, const float* f) {
        uint4 hi, lo;
        const float4 x0 = *reinterpret_cast<const float4*>(x + r * P + d), x1 = *reinterpret_cast<const float4*>(x + r * P + d + 4);
        const float4 f0 = *reinterpret_cast<const float4*>(f + b * DP + d), f1 = *reinterpret_cast<const float4*>(f + b * DP + d + 4);
        kd_split2<T>(x0.x * f0.x, x0.y * f0.y, hi.x, lo.x);
        kd_split2<T>(x0.z * f0.z, x0.w * f0.w, hi.y, lo.y);
        kd_split2<T>(x1.x * f1.x, x1.y * f1.y, hi.z, lo.z);
        kd_split2<T>(x1.z * f1.z, x1.w * f1.w, hi.w, lo.w);
        *reinterpret_cast<uint4*>(to) = hi;
        *reinterpret_cast<uint4*>(to + to_lo) = lo;
      };
      put(at + L.qg + panel1, L.plane1, sq, s_pre);
      put(at + L.kg + panel2, L.plane2, sa, s_suf);
      if constexpr (DELTA && !kSolveValues) put(at + L.w + panel1, L.plane1, sk, s_pre);
    }
  };
  if constexpr (!DELTA || kSolveValues) {
    store_q(tid >> 3, (tid & 7) * 4);
    store_rows(tid, kKdThreads);
  }
  if constexpr (DELTA && !kSolveValues) {
    // T: the inverses of its two diagonal blocks of 16 by forward substitution, a lane per column, while the others store; then
    // T_21 = -T_22 (beta K_21) T_11, a thread per entry
    constexpr int N = 16;
    float* sT = sQ;                                      // [32][36], once Q is stored
    float x[N];
    const int col = lane & (N - 1), blk = lane & N;
    if (warp == kKdThreads / 32 - 1) {
#pragma unroll
      for (int i = 0; i < N; i++) {
        float v = i == col ? 1.f : 0.f;
#pragma unroll
        for (int j = 0; j < i; j += 4) {
          const float4 f = *reinterpret_cast<const float4*>(sK + (blk + i) * 36 + blk + j);      // zero from the diagonal on
          v = fmaf(-f.x, x[j], v);
          if (j + 1 < i) v = fmaf(-f.y, x[j + 1], v);
          if (j + 2 < i) v = fmaf(-f.z, x[j + 2], v);
          if (j + 3 < i) v = fmaf(-f.w, x[j + 3], v);
        }
        x[i] = v;
      }
      reinterpret_cast<float*>(ops + L.beta)[lane] = s_beta[lane];
    } else {
      for (int i = tid; i < kKdChunk * 8; i += kKdThreads - 32) store_q(i >> 3, (i & 7) * 4);
      store_rows(tid, kKdThreads - 32);
    }
    __syncthreads();
    if (warp == kKdThreads / 32 - 1) {
#pragma unroll
      for (int i = 0; i < N; i++) sT[(blk + i) * 36 + blk + col] = x[i];
    }
    __syncthreads();
    const int i = tid >> 4, j = tid & 15;
    float m = 0.f;
#pragma unroll
    for (int n = 0; n < N; n++) m = fmaf(sK[(N + i) * 36 + n], sT[n * 36 + j], m);
    __syncthreads();
    sK[i * 36 + j] = m;                                  // the first block of K is no longer needed
    __syncthreads();
    m = 0.f;
#pragma unroll
    for (int n = 0; n < N; n++) m = fmaf(-sT[(N + i) * 36 + N + n], sK[n * 36 + j], m);
    auto put = [&](int r, int k, float v) {
      T hi, lo;
      kd_split<T>(v, hi, lo);
      uint8_t* at = ops + L.t + r * 128 + ((k * 2) ^ ((r & 7) << 4));
      *reinterpret_cast<T*>(at) = hi;
      *reinterpret_cast<T*>(at + kKdChunk * 128) = lo;
    };
    put(i, j, sT[i * 36 + j]);
    put(i, N + j, 0.f);
    put(N + i, j, m);
    put(N + i, N + j, sT[(N + i) * 36 + N + j]);
  } else if constexpr (DELTA) {
    // forward substitution with I + beta K, a thread per column: channels of A k, then value columns
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
    if (tid < DP) {
      float f = 1.f;
#pragma unroll
      for (int i = 0; i < kKdChunk; i++) {
        w[i] = sk[i * P + tid] * f;
        if (i % kKdBlock == kKdBlock - 1) f *= sb[i / kKdBlock * DP + tid];
      }
    }
    if (tid < DP || e_own < E) {
      solve(w);
      if (tid < DP) {
        T* at = reinterpret_cast<T*>(ops + L.w) + tid;
#pragma unroll
        for (int i = 0; i < kKdChunk; i++) {
          T hi, lo;
          kd_split<T>(-w[i], hi, lo);
          at[i * (DP + 8)] = hi;
          at[i * (DP + 8) + L.plane1 / 2] = lo;
        }
      } else store_u(e_own, w);
    }
#pragma unroll 1
    for (int e = tid + kKdThreads - DP; e < E; e += kKdThreads) { load_v(e, w); solve(w); store_u(e, w); }
  }
}

// ── scan, warp-level products (more than 128 channels) ──────────────────────
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
  constexpr KdOpsLayout L = kd_ops_layout(DP, DELTA);
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
    mbar_expect_tx(&full[c & 1], (uint32_t)L.bytes);
    kd_bulk_load(smem + (c & 1) * L.stride, p.ops + (sh * p.chunks + c) * L.stride, (uint32_t)L.bytes, &full[c & 1]);
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
    const T* qg = reinterpret_cast<const T*>(smem + sg * L.stride);
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

// ── scan on tcgen05 (up to 128 channels) ────────────────────────────────────
// A CTA: 128 value columns (lanes of tensor memory) of one head; two warps share a quarter of the lanes, each with half of the channels
// or tokens. Tensor memory columns: S^T in float32 [DP]; its high parts and remainders as A operand [DP]; two buffers of 128 columns,
// the products with high parts and remainders of the chunk's rows: (x | o | x' | o') with x = S (A k), otherwise (o | o').
// Per chunk:
//   warps 0 - 7    split S, fade it in place                        (after the update of the chunk before)
//   warp 12        (x | o) = S (A k | A q); without the delta rule o alone, u = v
//   warps 0 - 7    v behind its convolution, r = beta (v - x), split
//   warp 12        u = T r
//   warps 0 - 7    split u
//   warp 12        S += u (A_32 / A k), o += u Q
//   warps 8 - 11   o to memory, or through the head's norm and gate
// Warp 13 loads the chunks' operands. All waits are bounded.
constexpr int kd_stages(bool delta) { return delta ? 2 : 3; }      // chunks on their way; more shared memory would cost the delta rule's other loads their L1
constexpr int kKdStateWarps = 8, kKdMmaWarp = 12, kKdLoadWarp = 13, kKdScanThreads = 14 * 32, kKdHalf = kKdChunk / 2;
template <typename T, int DP, bool DELTA>
__global__ void __launch_bounds__(kKdScanThreads, 1) key_decay_scan_tc_kernel(const KdParams p, int fuse, int* status) {
  using namespace sm100;
  constexpr KdOpsLayout L = kd_ops_layout(DP, DELTA);
  constexpr uint32_t cS = 0, cA = 128, cO = 256, cR = cA + 64, cU = 64, kLo = L.rows1;      // cU: within a buffer; kLo: from a product to its remainder's
  constexpr int kSteps = DP / 16;
  extern __shared__ uint8_t smem_raw[];
  constexpr int kStages = kd_stages(DELTA);
  __shared__ uint64_t full[kStages], empty[kStages], s_ready, r_ready, u_ready, x_full, u_full, s_full, o_full[2], o_free[2], sums;
  __shared__ uint32_t tmem_slot;
  __shared__ float s_sum[2][4][kKdChunk];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, quarter = warp & 3, half = (warp >> 2) & 1;
  const int h = blockIdx.y, s = blockIdx.z, E = p.vdim, D = p.dim;
  const long long sh = (long long)s * p.heads + h;
  if (threadIdx.x == 0) {
    for (int i = 0; i < kStages; i++) { mbar_init(&full[i], 1); mbar_init(&empty[i], kKdStateWarps + 1); }
    for (int i = 0; i < 2; i++) { mbar_init(&o_full[i], 1); mbar_init(&o_free[i], 4); }
    mbar_init(&sums, 4);
    mbar_init(&s_ready, kKdStateWarps); mbar_init(&r_ready, kKdStateWarps); mbar_init(&u_ready, kKdStateWarps);
    mbar_init(&x_full, 1); mbar_init(&u_full, 1); mbar_init(&s_full, 1);
    mbar_fence_init();
  }
  if (warp == kKdMmaWarp) { tmem_alloc(&tmem_slot, 512); tmem_relinquish(); }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tm = tmem_slot;
  pdl_wait();
  pdl_trigger();
  const int e = (int)blockIdx.x * 128 + quarter * 32 + lane;         // value column of the threads that own one
  const uint32_t lanes = tm + ((uint32_t)(quarter * 32) << 16);
  if (warp == kKdLoadWarp) {
    if (lane == 0)
      for (int c = 0; c < p.chunks; c++) {
        const int st = c % kStages;
        if (!mbar_wait(&empty[st], (uint32_t)((c / kStages) & 1) ^ 1, status, 61)) break;
        mbar_expect_tx(&full[st], (uint32_t)L.bytes);
        kd_bulk_load(smem + st * L.stride, p.ops + (sh * p.chunks + c) * L.stride, (uint32_t)L.bytes, &full[st]);
      }
  } else if (warp == kKdMmaWarp) {
    if (lane == 0) {
      constexpr int fmt = std::is_same<T, __nv_bfloat16>::value ? 1 : 0;
      const uint32_t id_1 = make_idesc_f16(fmt, 0, 0, 128, 2 * L.rows1), id_2 = make_idesc_f16(fmt, 0, 0, 128, L.rows1);
      const uint32_t id_64 = make_idesc_f16(fmt, 0, 0, 128, 64), id_32 = make_idesc_f16(fmt, 0, 0, 128, 32), id_s = make_idesc_f16(fmt, 0, 1, 128, DP);
      const bool exact = !DELTA && p.taps == 0;                      // u is the stored v: no remainder
      for (int c = 0; c < p.chunks; c++) {
        const int st = c & 1, sg = c % kStages;
        const uint32_t ph = (uint32_t)(c & 1), ph2 = (uint32_t)((c >> 1) & 1), base = smem_u32(smem + sg * L.stride);
        const uint32_t buf = tm + cO + (uint32_t)(st * 128), acc_o = buf + (DELTA ? 32u : 0u), cu = buf + cU;
        if (!mbar_wait(&full[sg], (uint32_t)((c / kStages) & 1), status, 62) || !mbar_wait(&o_free[st], ph2 ^ 1, status, 63)) break;
        // a descriptor's address field counts 16-byte units: offsets are added to it
        const uint64_t d1 = make_smem_desc_sw128(base, 16, 1024), dq = d1 + (L.q >> 4), dt = d1 + (L.t >> 4), ds = make_smem_desc_sw128(base + L.kg, kKdChunk * 128, 1024);
        auto rows_product = [&](int k) {                             // high parts with the rows and their remainders side by side, remainders with the rows
          const uint64_t d = d1 + (((k >> 2) * 2 * L.plane1 + (k & 3) * 32) >> 4);
          mma_f16_ts(buf, tm + cA + (uint32_t)(k * 8), d, id_1, k > 0 ? 1u : 0u);
          mma_f16_ts(buf, tm + cA + (uint32_t)(DP / 2 + k * 8), d, id_2, 1u);
        };
        auto state_product = [&]() {                                 // high x high, remainder x high, high x remainder
#pragma unroll
          for (int part = 0; part < 3; part++) {
            if (part == 1 && exact) continue;
#pragma unroll
            for (int k = 0; k < kKdChunk / 16; k++)
              mma_f16_ts(tm + cS, cu + (uint32_t)((part == 1 ? 16 : 0) + k * 8), ds + (((part == 2 ? L.plane2 : 0) + k * 2048) >> 4), id_s, 1u);
          }
          mma_commit(&s_full);
        };
        if constexpr (DELTA) {
          if (!mbar_wait(&s_ready, ph, status, 64)) break;
          tc_fence_after_sync();
#pragma unroll
          for (int k = 0; k < kSteps; k++) rows_product(k);
          mma_commit(&x_full);
          if (!mbar_wait(&r_ready, ph, status, 65)) break;
          tc_fence_after_sync();
          mma_f16_ts(tm + cA, tm + cR, dt, id_64, 0u);               // the operand S is no longer needed: u and its remainder take its place
          mma_f16_ts(tm + cA, tm + cR + 8, dt + 2, id_64, 1u);
          mma_f16_ts(tm + cA, tm + cR + 16, dt, id_32, 1u);
          mma_f16_ts(tm + cA, tm + cR + 24, dt + 2, id_32, 1u);
          mma_commit(&u_full);
          if (!mbar_wait(&u_ready, ph, status, 73)) break;
          tc_fence_after_sync();
          state_product();
        } else {
          if (!mbar_wait(&s_ready, ph, status, 64)) break;
          tc_fence_after_sync();
          state_product();                                           // needs no more than u: ahead of the rows, which read the split copy of S
#pragma unroll
          for (int k = 0; k < kSteps; k++) rows_product(k);
          mma_commit(&x_full);
        }
#pragma unroll
        for (int part = 0; part < 3; part++) {
          if (part == 1 && exact) continue;
#pragma unroll
          for (int k = 0; k < kKdChunk / 16; k++)
            mma_f16_ts(acc_o, cu + (uint32_t)((part == 1 ? 16 : 0) + k * 8), dq + (((part == 2 ? 64 : 0) + k * 32) >> 4), id_32, 1u);
        }
        mma_commit(&o_full[st]);
        mma_commit(&empty[sg]);
      }
    }
  } else if (warp < kKdStateWarps) {
    constexpr int G = DP / 16;                                       // pieces of 16 channels, every other one is this warp's
    const int ec = min(e, E - 1), vcol = p.v_off + h * E + ec, vch = 2 * p.qk_heads * D + h * E + ec, tb = half * kKdHalf;
    const T* base = reinterpret_cast<const T*>(p.proj) + (long long)s * p.T * p.ld;
    const T* ring = p.ring_of<T>(s);
    const int pos = p.pos[s];
    float taps[kKdTaps];
#pragma unroll
    for (int i = 0; i < kKdTaps; i++) taps[i] = i == kKdTaps - 1 ? 1.f : 0.f;
    if (p.taps && p.taps <= kKdTaps) kd_taps(p, vch, taps);
    float* S = p.state(s) + (long long)h * D * E;
    uint32_t x[16];
#pragma unroll 1
    for (int g = half; g < G; g += 2) {
      const float* row = S + (long long)g * 16 * E + e;
#pragma unroll
      for (int i = 0; i < 16; i++, row += E) x[i] = g * 16 + i < D && e < E ? __float_as_uint(*row) : 0u;
      tmem_st_32x16(lanes + cS + (uint32_t)(g * 16), x);
    }
    tmem_st_wait();
    bool ok = true;
    auto split = [&](const float (&v)[16], uint32_t at, uint32_t lo_off) {
      uint32_t hi[8], lo[8];
#pragma unroll
      for (int i = 0; i < 8; i++) kd_split2<T, !DELTA>(v[2 * i], v[2 * i + 1], hi[i], lo[i]);
      tmem_st_32x8(at, hi);
      tmem_st_32x8(at + lo_off, lo);
    };
    auto arrive = [&](uint64_t* bar) {
      tmem_st_wait();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar);
    };
    // this thread's raw values of a chunk and the ones before them, requested a chunk ahead
    uint32_t raw[kKdHalf + kKdTaps - 1];
    auto request = [&](int t0) {
      const T* src = base + (long long)(t0 - (kKdTaps - 1)) * p.ld + vcol;
      if (t0 >= kKdTaps - 1 && t0 + kKdHalf <= p.T) {
#pragma unroll
        for (int i = 0; i < kKdHalf + kKdTaps - 1; i++, src += p.ld) raw[i] = kd_bits<T>(src);
      } else {
#pragma unroll
        for (int i = 0; i < kKdHalf + kKdTaps - 1; i++) {
          const int t = t0 - (kKdTaps - 1) + i;
          raw[i] = t >= p.T || (t < 0 && -t >= p.taps) ? 0u : t >= 0 ? kd_bits<T>(src + (long long)i * p.ld) : kd_round_bits<T>(kd_raw<T>(p, base, ring, pos, t, vcol, vch));
        }
      }
    };
    request(tb);
    for (int c = 0; c < p.chunks; c++) {
      const int st = c & 1, sg = c % kStages, t0 = c * kKdChunk + tb;
      const uint32_t ph = (uint32_t)(c & 1), buf = lanes + cO + (uint32_t)(st * 128);
      float v[kKdHalf];
      auto values = [&]() {
        if (p.taps == 0) {
#pragma unroll
          for (int i = 0; i < kKdHalf; i++) v[i] = kd_value<T>(raw[i + kKdTaps - 1]);
        } else if (p.taps <= kKdTaps) {
#pragma unroll
          for (int i = 0; i < kKdHalf; i++) {
            float y = 0.f;
#pragma unroll
            for (int n = 0; n < kKdTaps; n++) y = fmaf(taps[n], kd_value<T>(raw[i + n]), y);
            v[i] = kd_silu_fast(y);
          }
        } else {
#pragma unroll 1
          for (int i = 0; i < kKdHalf; i++) {
            const float y = t0 + i < p.T ? kd_input<T>(p, base, ring, pos, t0 + i, vcol, vch) : 0.f;
#pragma unroll
            for (int j = 0; j < kKdHalf; j++) if (j == i) v[j] = y;
          }
        }
        if (t0 + kKdHalf > p.T || e >= E) {
#pragma unroll
          for (int i = 0; i < kKdHalf; i++) if (t0 + i >= p.T || e >= E) v[i] = 0.f;
        }
        if (c + 1 < p.chunks) request(t0 + kKdChunk);
      };
      ok = __all_sync(0xffffffffu, mbar_wait(&full[sg], (uint32_t)((c / kStages) & 1), status, 66) && (c == 0 || mbar_wait(&s_full, ph ^ 1, status, 67)));
      if (!ok) break;
      tc_fence_after_sync();
      const float4* decay = reinterpret_cast<const float4*>(smem + sg * L.stride + L.decay);
      uint32_t next[16];                                             // on its way while a piece is split
      tmem_ld_32x16(lanes + cS + (uint32_t)(half * 16), next);
      if (!DELTA && c > 0) {                                         // the copy of S is still an operand of the last rows
        ok = __all_sync(0xffffffffu, mbar_wait(&x_full, ph ^ 1, status, 72));
        if (!ok) break;
        tc_fence_after_sync();
      }
#pragma unroll(DELTA ? 1 : 8)
      for (int n = 0; n < (G + 1) / 2; n++) {
        const int g = 2 * n + half;
        if (G % 2 && g >= G) break;
        tmem_ld_wait();
        float y[16];
#pragma unroll
        for (int i = 0; i < 16; i++) y[i] = __uint_as_float(next[i]);
        if (g + 2 < G) tmem_ld_32x16(lanes + cS + (uint32_t)((g + 2) * 16), next);
        split(y, lanes + cA + (uint32_t)(g * 8), DP / 2);
#pragma unroll
        for (int i = 0; i < 4; i++) {
          const float4 f = decay[g * 4 + i];
          if constexpr (DELTA) {
            x[4 * i] = __float_as_uint(y[4 * i] * f.x); x[4 * i + 1] = __float_as_uint(y[4 * i + 1] * f.y);
            x[4 * i + 2] = __float_as_uint(y[4 * i + 2] * f.z); x[4 * i + 3] = __float_as_uint(y[4 * i + 3] * f.w);
          } else {
            const uint64_t a = mul_f32x2(pack_f32x2(y[4 * i], y[4 * i + 1]), pack_f32x2(f.x, f.y)), b = mul_f32x2(pack_f32x2(y[4 * i + 2], y[4 * i + 3]), pack_f32x2(f.z, f.w));
            x[4 * i] = (uint32_t)a; x[4 * i + 1] = (uint32_t)(a >> 32); x[4 * i + 2] = (uint32_t)b; x[4 * i + 3] = (uint32_t)(b >> 32);
          }
        }
        tmem_st_32x16(lanes + cS + (uint32_t)(g * 16), x);
      }
      if constexpr (!DELTA) {
        values();
        split(v, buf + cU + (uint32_t)(half * 8), 16);               // its last reader was this buffer's o, two chunks ago
        arrive(&s_ready);
        if (lane == 0) mbar_arrive(&empty[sg]);
      } else {
        arrive(&s_ready);
        values();
        const float4* beta = reinterpret_cast<const float4*>(smem + sg * L.stride + L.beta) + tb / 4;
        float b[kKdHalf];
#pragma unroll
        for (int i = 0; i < kKdHalf / 4; i++) { const float4 f = beta[i]; b[4 * i] = f.x; b[4 * i + 1] = f.y; b[4 * i + 2] = f.z; b[4 * i + 3] = f.w; }
        __syncwarp();
        if (lane == 0) mbar_arrive(&empty[sg]);
        uint32_t y[16];
        ok = __all_sync(0xffffffffu, mbar_wait(&x_full, ph, status, 68));
        if (!ok) break;
        tc_fence_after_sync();
        tmem_ld_32x16(buf + (uint32_t)tb, x);
        tmem_ld_32x16(buf + kLo + (uint32_t)tb, y);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < kKdHalf; i++) v[i] = b[i] * (v[i] - (__uint_as_float(x[i]) + __uint_as_float(y[i])));
        split(v, lanes + cR + (uint32_t)(half * 8), 16);
        arrive(&r_ready);
        ok = __all_sync(0xffffffffu, mbar_wait(&u_full, ph, status, 74));
        if (!ok) break;
        tc_fence_after_sync();
        tmem_ld_32x16(lanes + cA + (uint32_t)tb, x);
        tmem_ld_32x16(lanes + cA + 32u + (uint32_t)tb, y);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < kKdHalf; i++) v[i] = __uint_as_float(x[i]) + __uint_as_float(y[i]);
        split(v, buf + cU + (uint32_t)(half * 8), 16);
        arrive(&u_ready);
      }
    }
    ok = ok && __all_sync(0xffffffffu, mbar_wait(&s_full, (uint32_t)((p.chunks - 1) & 1), status, 69));
    if (ok) {
      tc_fence_after_sync();
#pragma unroll 1
      for (int g = half; g < G; g += 2) {
        tmem_ld_32x16(lanes + cS + (uint32_t)(g * 16), x);
        tmem_ld_wait();
        float* row = S + (long long)g * 16 * E + e;
#pragma unroll
        for (int i = 0; i < 16; i++, row += E) if (g * 16 + i < D && e < E) *row = __uint_as_float(x[i]);
      }
      tc_fence_before_sync();
    }
  } else {
    const float nw = e < E ? p.norm[e] : 0.f;
    for (int c = 0; c < p.chunks; c++) {
      const int st = c & 1, t0 = c * kKdChunk, nt = min(kKdChunk, p.T - t0);
      const long long row0 = (long long)s * p.T + t0;
      const bool whole = __all_sync(0xffffffffu, e < E) && nt == kKdChunk;
      uint32_t gate[kKdChunk];
      if (fuse) {
        const T* g = p.gate ? reinterpret_cast<const T*>(p.gate) + row0 * p.gate_ld + (long long)h * E + e : reinterpret_cast<const T*>(p.proj) + row0 * p.ld + p.g_off + (long long)h * E + e;
        const long long ld = p.gate ? p.gate_ld : p.ld;
        if (whole) {
#pragma unroll
          for (int i = 0; i < kKdChunk; i++, g += ld) gate[i] = kd_bits<T>(g);
        } else {
#pragma unroll
          for (int i = 0; i < kKdChunk; i++, g += ld) gate[i] = e < E && i < nt ? kd_bits<T>(g) : 0u;
        }
      }
      if (!__all_sync(0xffffffffu, mbar_wait(&o_full[st], (uint32_t)((c >> 1) & 1), status, 70))) break;
      tc_fence_after_sync();
      float o[kKdChunk];
#pragma unroll
      for (int n = 0; n < 2; n++) {
        uint32_t x[16], y[16];
        const uint32_t at = lanes + cO + (uint32_t)(st * 128 + (DELTA ? 32 : 0) + n * kKdHalf);
        tmem_ld_32x16(at, x);
        tmem_ld_32x16(at + kLo, y);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < kKdHalf; i++) o[n * kKdHalf + i] = __uint_as_float(x[i]) + __uint_as_float(y[i]);
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&o_free[st]);
      if (!fuse) {
        float* O = p.o + (row0 * p.heads + h) * E + e;
#pragma unroll
        for (int i = 0; i < kKdChunk; i++) if (i < nt && e < E) O[(long long)i * p.heads * E] = o[i];
        continue;
      }
      // sums of squares over the value columns: after five halvings lane t holds token t's
      float v[kKdHalf];
      {
        const bool up = lane & 16;
#pragma unroll
        for (int i = 0; i < kKdHalf; i++) {
          const float a = o[i] * o[i], b = o[i + kKdHalf] * o[i + kKdHalf], other = __shfl_xor_sync(0xffffffffu, up ? a : b, 16);
          v[i] = (up ? b : a) + other;
        }
      }
#pragma unroll
      for (int w = 8; w > 0; w >>= 1) {
        const bool up = lane & w;
#pragma unroll
        for (int i = 0; i < w; i++) {
          const float other = __shfl_xor_sync(0xffffffffu, up ? v[i] : v[i + w], w);
          v[i] = (up ? v[i + w] : v[i]) + other;
        }
      }
      s_sum[st][quarter][lane] = v[0];
      __syncwarp();
      if (lane == 0) mbar_arrive(&sums);
      if (!__all_sync(0xffffffffu, mbar_wait(&sums, (uint32_t)st, status, 71))) break;
      const float rs = 1.0f / sqrtf((s_sum[st][0][lane] + s_sum[st][1][lane] + s_sum[st][2][lane] + s_sum[st][3][lane]) / (float)E + p.eps);
      T* out = reinterpret_cast<T*>(p.y) + row0 * p.y_ld + (long long)h * E + e;
      T res[kKdChunk];
#pragma unroll
      for (int i = 0; i < kKdChunk; i++) {
        res[i] = Cvt<T>::from(o[i] * (__shfl_sync(0xffffffffu, rs, i) * nw) * kd_gate_fast(p, kd_value<T>(gate[i])));
      }
      if (whole) {
#pragma unroll
        for (int i = 0; i < kKdChunk; i++, out += p.y_ld) *out = res[i];
      } else {
#pragma unroll
        for (int i = 0; i < kKdChunk; i++, out += p.y_ld) if (e < E && i < nt) *out = res[i];
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  if (warp == kKdMmaWarp) tmem_dealloc(tm, 512);
}

// ── finish: norm and gate of the heads' outputs, a warp each ────────────────
// REG: float4 pieces of a head a lane keeps; 0: any width and alignment, read twice
constexpr int kKdItems = 2;            // heads a warp works on
template <typename T, int REG>
__global__ void __launch_bounds__(256) key_decay_finish_kernel(const KdParams p) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31, E = p.vdim;
  const long long items = (long long)p.n_seq * p.T * p.heads, i0 = ((long long)blockIdx.x * 8 + (threadIdx.x >> 5)) * kKdItems;
  auto gate_of = [&](long long i) {
    const long long r = (uint32_t)i / (uint32_t)p.heads, c = (long long)((uint32_t)i % (uint32_t)p.heads) * E;
    return p.gate ? reinterpret_cast<const T*>(p.gate) + r * p.gate_ld + c : reinterpret_cast<const T*>(p.proj) + r * p.ld + p.g_off + c;
  };
  auto out_of = [&](long long i) { return reinterpret_cast<T*>(p.y) + (long long)((uint32_t)i / (uint32_t)p.heads) * p.y_ld + (long long)((uint32_t)i % (uint32_t)p.heads) * E; };
  if constexpr (REG > 0) {
    float4 v[kKdItems][REG];
    uint2 z[kKdItems][REG];
#pragma unroll
    for (int n = 0; n < kKdItems; n++)
#pragma unroll
      for (int q = 0; q < REG; q++) {
        const int e = (lane + 32 * q) * 4;
        v[n][q] = make_float4(0.f, 0.f, 0.f, 0.f);
        z[n][q] = make_uint2(0u, 0u);
        if (i0 + n < items && e < E) { v[n][q] = __ldcs(reinterpret_cast<const float4*>(p.o + (i0 + n) * E + e)); z[n][q] = *reinterpret_cast<const uint2*>(gate_of(i0 + n) + e); }
      }
#pragma unroll
    for (int n = 0; n < kKdItems; n++) {
      float sq = 0.f;
#pragma unroll
      for (int q = 0; q < REG; q++) sq = fmaf(v[n][q].x, v[n][q].x, fmaf(v[n][q].y, v[n][q].y, fmaf(v[n][q].z, v[n][q].z, fmaf(v[n][q].w, v[n][q].w, sq))));
      const float rs = 1.0f / sqrtf(warp_sum(sq) / (float)E + p.eps);
#pragma unroll
      for (int q = 0; q < REG; q++) {
        const int e = (lane + 32 * q) * 4;
        if (i0 + n >= items || e >= E) continue;
        const float4 x = v[n][q], w = __ldg(reinterpret_cast<const float4*>(p.norm + e));
        const T* gv = reinterpret_cast<const T*>(&z[n][q]);
        uint2 out;
        out.x = pack2_t<T>(x.x * rs * w.x * kd_gate_fast(p, Cvt<T>::to(gv[0])), x.y * rs * w.y * kd_gate_fast(p, Cvt<T>::to(gv[1])));
        out.y = pack2_t<T>(x.z * rs * w.z * kd_gate_fast(p, Cvt<T>::to(gv[2])), x.w * rs * w.w * kd_gate_fast(p, Cvt<T>::to(gv[3])));
        *reinterpret_cast<uint2*>(out_of(i0 + n) + e) = out;
      }
    }
  } else {
    for (long long i = i0; i < i0 + kKdItems && i < items; i++) {
      const float* o = p.o + i * E;
      const T* g = gate_of(i);
      T* y = out_of(i);
      float sq = 0.f;
      for (int e = lane; e < E; e += 32) sq = fmaf(o[e], o[e], sq);
      const float rs = 1.0f / sqrtf(warp_sum(sq) / (float)E + p.eps);
      for (int e = lane; e < E; e += 32) y[e] = Cvt<T>::from(o[e] * rs * p.norm[e] * kd_gate_fast(p, Cvt<T>::to(g[e])));
    }
  }
}

// ── host ────────────────────────────────────────────────────────────────────
template <typename T, int DP, bool DELTA>
static cudaError_t launch_kd(cudaStream_t s, const KdParams& p) {
  constexpr KdOpsLayout L = kd_ops_layout(DP, DELTA);
  constexpr size_t prep = ((size_t)3 * kKdChunk * (DP + 4) + kKdBlocks * DP + 2 * kKdChunk * 36 + 3 * kKdChunk + DP + (2 * kKdBlocks * DP > 4 * 768 ? 2 * kKdBlocks * DP : 4 * 768)) * sizeof(float);
  constexpr size_t scan = kd_tc(DP) ? kd_stages(DELTA) * (size_t)L.stride + 1024 : 2 * (size_t)L.stride;
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(key_decay_prepare_kernel<T, DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)prep);
    if (e == cudaSuccess) {
      if constexpr (kd_tc(DP)) e = cudaFuncSetAttribute(key_decay_scan_tc_kernel<T, DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan);
      else e = cudaFuncSetAttribute(key_decay_scan_kernel<T, DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan);
    }
    if (e != cudaSuccess) return e;
    attr = true;
  }
  cudaError_t e = launch_pdl(key_decay_prepare_kernel<T, DP, DELTA>, dim3((unsigned)p.chunks, (unsigned)p.heads, (unsigned)p.n_seq), dim3(kKdThreads), prep, s, p);
  if (e != cudaSuccess) return e;
  if constexpr (kd_tc(DP)) {
    return launch_pdl(key_decay_scan_tc_kernel<T, DP, DELTA>, dim3((unsigned)((p.vdim + 127) / 128), (unsigned)p.heads, (unsigned)p.n_seq), dim3(kKdScanThreads), scan, s, p, kd_fused(p.dp, p.vdim) ? 1 : 0,
                      matmul_status_word());
  } else {
    // value columns per CTA: up to 128, fewer where that leaves SMs without work
    int warps = std::min(8, (p.vdim + 15) / 16);
    while (warps > 2 && (long long)p.n_seq * p.heads * ((p.vdim + 16 * warps - 1) / (16 * warps)) < sm_count()) warps = (warps + 1) / 2;
    return launch_pdl(key_decay_scan_kernel<T, DP, DELTA>, dim3((unsigned)((p.vdim + 16 * warps - 1) / (16 * warps)), (unsigned)p.heads, (unsigned)p.n_seq), dim3((unsigned)warps * 32), scan, s, p,
                      matmul_status_word());
  }
}
template <typename T, bool DELTA>
static cudaError_t launch_kd_dp(cudaStream_t s, const KdParams& p) {
  switch (p.dp) {
    case 32: return launch_kd<T, 32, DELTA>(s, p);
    case 64: return launch_kd<T, 64, DELTA>(s, p);
    case 96: return launch_kd<T, 96, DELTA>(s, p);
    case 128: return launch_kd<T, 128, DELTA>(s, p);
    case 192: return launch_kd<T, 192, DELTA>(s, p);
    default: return launch_kd<T, 256, DELTA>(s, p);
  }
}
template <typename T>
static Status launch_chunked(cudaStream_t s, const KdParams& p) {
  cudaError_t e = p.delta ? launch_kd_dp<T, true>(s, p) : launch_kd_dp<T, false>(s, p);
  if (e != cudaSuccess || kd_fused(p.dp, p.vdim)) return cuda_status(e, "key decay (chunked)");
  const unsigned blocks = (unsigned)(((long long)p.n_seq * p.T * p.heads + 8 * kKdItems - 1) / (8 * kKdItems));
  const bool vec = p.vdim % 4 == 0 && p.y_ld % 4 == 0 && aligned16(p.y) && aligned16(p.norm) && (p.gate ? p.gate_ld % 4 == 0 : p.ld % 4 == 0 && p.g_off % 4 == 0 && aligned16(p.proj));
  if (vec && p.vdim <= 128) e = launch_pdl(key_decay_finish_kernel<T, 1>, dim3(blocks), dim3(256), 0, s, p);
  else if (vec && p.vdim <= 256) e = launch_pdl(key_decay_finish_kernel<T, 2>, dim3(blocks), dim3(256), 0, s, p);
  else e = launch_pdl(key_decay_finish_kernel<T, 0>, dim3(blocks), dim3(256), 0, s, p);
  return cuda_status(e, "key decay (chunked)");
}

}}  // namespace ag::k
