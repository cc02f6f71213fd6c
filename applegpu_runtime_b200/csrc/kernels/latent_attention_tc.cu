// Prompt attention of the latent kind on tcgen05: query / key rows of up to 256 entries made of an unrotated part per head
// and a rotated part whose keys all heads share, values of up to 256, keys behind any number of cached tokens.
//
// Built like attention_tc.cu, for wider heads. A CTA takes NT = 2 neighbouring tiles of 128 query rows of one head (NT = 1
// above 128 value columns) and walks their keys in blocks of 64, every K and V block loaded once for both tiles: warp 0
// loads (TMA, 64-column panels: the unrotated part, zero-filled past its end, then the rotated one, each from its own
// tensor), warp 1 issues the MMAs, four softmax warps per tile hold one query row per thread. Scores of the next two
// blocks are issued while the softmax works, the two tiles' softmax groups keep the tensor pipe busy in turns. The weights are
// float32 values that enter the P V product as the sum of two 16-bit numbers (high part and remainder, in the two halves of
// the score buffer they came from), so the product does not round them to the storage type. All waits are bounded.
#include "common.cuh"
#include "seq_kernels.h"
#include "sm100.cuh"
#include "tc_math.cuh"
#include <cuda.h>
#include <type_traits>

namespace ag { namespace k {

using namespace ag::sm100;

Status make_map(CUtensorMap* out, DType dt, const void* ptr, uint64_t inner, uint64_t rows, uint64_t nbi, uint64_t nbo,
                uint64_t row_stride, uint64_t bi_stride, uint64_t bo_stride, uint32_t b0, uint32_t b1);

constexpr int kLtQ = 128, kLtKeys = 64, kLtPanel = 64, kLtMaxStages = 4;
constexpr int kLtQPanel = kLtQ * kLtPanel * 2, kLtKPanel = kLtKeys * kLtPanel * 2;
constexpr int kLtSmemMax = 226 * 1024;
constexpr float kLtRescaleLog2 = 8.0f;      // see attention_tc.cu: growth of the maximum that is carried without rescaling

struct LatTcParams {
  void* y;
  long long y_b, y_h, y_t;
  int heads, bh, tq, past, pairs;           // pairs: query tile groups per head
  int dim, rot, vdim, pd, pr, pv, stages;   // panels of the unrotated, rotated and value columns
  int y_vec;
  float scale_log2;
  int* status;
};

// 16-wide MMA steps that panel `c` of a part of `n` columns needs
__device__ __forceinline__ int lt_steps(int n, int c) { const int left = n - c * kLtPanel; return left >= kLtPanel ? 4 : (left + 15) / 16; }

template <typename T, int NT>
__global__ void __launch_bounds__(64 + NT * 128, 1)
latent_attention_tc_kernel(const __grid_constant__ CUtensorMap mq, const __grid_constant__ CUtensorMap mqr, const __grid_constant__ CUtensorMap mk,
                           const __grid_constant__ CUtensorMap mkr, const __grid_constant__ CUtensorMap mv, const LatTcParams p) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t q_full[NT], k_full[kLtMaxStages], k_empty[kLtMaxStages], v_full[kLtMaxStages], v_empty[kLtMaxStages], s_full[NT][2], p_full[NT][2], o_full[NT][2];
  __shared__ uint32_t tmem_base_slot;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int qp = p.pd + p.pr;
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + NT * qp * kLtQPanel;
  uint8_t* sV = sK + p.stages * qp * kLtKPanel;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < kLtMaxStages; s++) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1); }
    for (int t = 0; t < NT; t++) {
      mbar_init(&q_full[t], 1);
      for (int s = 0; s < 2; s++) { mbar_init(&s_full[t][s], 1); mbar_init(&p_full[t][s], 4); mbar_init(&o_full[t][s], 1); }
    }
    mbar_fence_init();
    prefetch_tmap(&mq); prefetch_tmap(&mqr); prefetch_tmap(&mk); prefetch_tmap(&mkr); prefetch_tmap(&mv);
  }
  if (warp == 1) { tmem_alloc(&tmem_base_slot, 512); tmem_relinquish(); }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = tmem_base_slot;
  // columns: the score buffers (two of 64 per tile), then the outputs (128 columns per tile, 256 for a single tile)
  auto tmem_s = [&](int t, int b) { return tmem_base + (uint32_t)((t * 2 + b) * kLtKeys); };
  auto tmem_o = [&](int t) { return tmem_base + (uint32_t)(NT * 2 * kLtKeys + t * 128); };
  pdl_wait();
  pdl_trigger();

  // longest tiles first
  const int g = (int)blockIdx.x / p.bh, bh = (int)blockIdx.x % p.bh;
  const int b = bh / p.heads, h = bh % p.heads;
  const int q0 = (p.pairs - 1 - g) * NT * kLtQ;
  const int tk = p.past + p.tq;
  int nb[NT], n_max = 0;
#pragma unroll
  for (int t = 0; t < NT; t++) {
    const int first = q0 + t * kLtQ;
    nb[t] = first < p.tq ? (min(tk, p.past + first + kLtQ) + kLtKeys - 1) / kLtKeys : 0;
    n_max = max(n_max, nb[t]);
  }

  if (warp == 0) {
    if (lane == 0) {
      bool ok = true;
      for (int t = 0; t < NT; t++) {
        if (nb[t] == 0) continue;
        mbar_expect_tx(&q_full[t], (uint32_t)(qp * kLtQPanel));
        uint8_t* dst = sQ + t * qp * kLtQPanel;
        for (int c = 0; c < p.pd; c++) tma_load_4d(dst + c * kLtQPanel, &mq, &q_full[t], c * kLtPanel, q0 + t * kLtQ, h, b);
        for (int c = 0; c < p.pr; c++) tma_load_4d(dst + (p.pd + c) * kLtQPanel, &mqr, &q_full[t], c * kLtPanel, q0 + t * kLtQ, h, b);
      }
      for (int j = 0; j < n_max && ok; j++) {
        const int st = j % p.stages;
        const uint32_t ph = (uint32_t)((j / p.stages) & 1);
        if (!mbar_wait(&k_empty[st], ph ^ 1, p.status, 32)) { ok = false; break; }
        mbar_expect_tx(&k_full[st], (uint32_t)(qp * kLtKPanel));
        uint8_t* dk = sK + st * qp * kLtKPanel;
        for (int c = 0; c < p.pd; c++) tma_load_4d(dk + c * kLtKPanel, &mk, &k_full[st], c * kLtPanel, j * kLtKeys, h, b);
        for (int c = 0; c < p.pr; c++) tma_load_4d(dk + (p.pd + c) * kLtKPanel, &mkr, &k_full[st], c * kLtPanel, j * kLtKeys, 0, b);
        if (!mbar_wait(&v_empty[st], ph ^ 1, p.status, 33)) { ok = false; break; }
        mbar_expect_tx(&v_full[st], (uint32_t)(p.pv * kLtKPanel));
        uint8_t* dv = sV + st * p.pv * kLtKPanel;
        for (int c = 0; c < p.pv; c++) tma_load_4d(dv + c * kLtKPanel, &mv, &v_full[st], c * kLtPanel, j * kLtKeys, h, b);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr int fmt = std::is_same<T, __nv_bfloat16>::value ? 1 : 0;
      const uint32_t idesc_s = make_idesc_f16(fmt, 0, 0, kLtQ, kLtKeys);
      const uint32_t idesc_o = make_idesc_f16(fmt, 0, 1, kLtQ, (p.vdim + 15) / 16 * 16);
      bool ok = true;
      // scores of block j for every tile that sees it
      auto issue_s = [&](int j) -> bool {
        if (j >= n_max) return true;
        const int st = j % p.stages;
        if (!mbar_wait(&k_full[st], (uint32_t)((j / p.stages) & 1), p.status, 34)) return false;
        for (int t = 0; t < NT; t++) {
          if (j >= nb[t]) continue;
          if (j == 0 && !mbar_wait(&q_full[t], 0, p.status, 35)) return false;
          tc_fence_after_sync();
          uint32_t acc = 0;
          for (int c = 0; c < qp; c++) {
            const uint32_t a = smem_u32(sQ + (t * qp + c) * kLtQPanel), bb = smem_u32(sK + (st * qp + c) * kLtKPanel);
            const int steps = c < p.pd ? lt_steps(p.dim, c) : lt_steps(p.rot, c - p.pd);
            for (int kk = 0; kk < steps; kk++, acc = 1)
              mma_f16_ss(tmem_s(t, j & 1), make_smem_desc_sw128(a + kk * 32, 16, 1024), make_smem_desc_sw128(bb + kk * 32, 16, 1024), idesc_s, acc);
          }
          mma_commit(&s_full[t][j & 1]);
        }
        mma_commit(&k_empty[st]);
        return true;
      };
      ok = issue_s(0) && issue_s(1);
      for (int j = 0; j < n_max && ok; j++) {
        const int st = j % p.stages;
        if (!mbar_wait(&v_full[st], (uint32_t)((j / p.stages) & 1), p.status, 36)) { ok = false; break; }
        for (int t = 0; t < NT && ok; t++) {
          if (j >= nb[t]) continue;
          if (!mbar_wait(&p_full[t][j & 1], (uint32_t)((j >> 1) & 1), p.status, 37)) { ok = false; break; }
          tc_fence_after_sync();
          const uint32_t bb = smem_u32(sV + st * p.pv * kLtKPanel);
#pragma unroll
          for (int part = 0; part < 2; part++)
#pragma unroll
            for (int kk = 0; kk < kLtKeys / 16; kk++)
              mma_f16_ts(tmem_o(t), tmem_s(t, j & 1) + (uint32_t)(part * 32 + kk * 8), make_smem_desc_sw128(bb + kk * 2048, kLtKPanel, 1024), idesc_o,
                         (j > 0 || part > 0 || kk > 0) ? 1u : 0u);
          mma_commit(&o_full[t][j & 1]);
        }
        if (!ok) break;
        mma_commit(&v_empty[st]);
        ok = issue_s(j + 2);
      }
    }
  } else {
    const int t = (warp - 2) >> 2;
    const int quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(quarter * 32) << 16;
    const int row = q0 + t * kLtQ + r;
    const float sc = p.scale_log2;
    const int n_blocks = t == 0 ? nb[0] : nb[NT - 1];
    const int o_cols = (p.vdim + 31) / 32;
    float m_ref = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int j = 0; j < n_blocks; j++) {
      const int sb = j & 1;
      if (!__all_sync(0xffffffffu, mbar_wait(&s_full[t][sb], (uint32_t)((j >> 1) & 1), p.status, 38))) { ok = false; break; }
      tc_fence_after_sync();
      uint32_t s0[32], s1[32];
      tmem_ld_32x32(tmem_s(t, sb) + lane_addr, s0);
      tmem_ld_32x32(tmem_s(t, sb) + lane_addr + 32u, s1);
      tmem_ld_wait();
      const int lim = min(min(tk, p.past + row + 1) - j * kLtKeys, kLtKeys);      // columns of the block this row sees
      if (!__all_sync(0xffffffffu, lim >= kLtKeys)) {
#pragma unroll
        for (int e = 0; e < 32; e++) {
          if (e >= lim) s0[e] = 0xff800000u;
          if (32 + e >= lim) s1[e] = 0xff800000u;
        }
      }
      float m_blk;
      {
        auto sv = [&](int i) { return __uint_as_float(i < 32 ? s0[i] : s1[i - 32]); };
        float mc[4] = {sv(0), sv(1), sv(2), sv(3)};
#pragma unroll
        for (int i = 0; i < 30; i++) mc[i & 3] = max3_f32(mc[i & 3], sv(4 + 2 * i), sv(5 + 2 * i));
        m_blk = fmaxf(max3_f32(mc[0], mc[1], mc[2]), mc[3]);
      }
      const float m_cand = fmaxf(m_ref, m_blk * sc);
      const bool moves = (m_cand - m_ref > kLtRescaleLog2) || (m_ref == -INFINITY && m_cand != -INFINITY);
      float alpha = 1.0f;
      const bool any_moves = __any_sync(0xffffffffu, moves);
      if (any_moves && moves) { alpha = ex2_approx(m_ref - m_cand); m_ref = m_cand; }
      if (j > 0 && any_moves) {
        if (!__all_sync(0xffffffffu, mbar_wait(&o_full[t][(j - 1) & 1], (uint32_t)(((j - 1) >> 1) & 1), p.status, 39))) { ok = false; break; }
        tc_fence_after_sync();
        for (int c = 0; c < o_cols; c++) {
          uint32_t ov[32];
          tmem_ld_32x32(tmem_o(t) + lane_addr + (uint32_t)(c * 32), ov);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 32; e++) ov[e] = __float_as_uint(__uint_as_float(ov[e]) * alpha);
          tmem_st_32x32(tmem_o(t) + lane_addr + (uint32_t)(c * 32), ov);
        }
        tmem_st_wait();
      }
      l_run *= alpha;
      const float m_use = (m_ref == -INFINITY) ? 0.f : m_ref;
      const uint64_t sc2 = pack_f32x2(sc, sc), nm2 = pack_f32x2(-m_use, -m_use);
      uint64_t acc[2] = {0ull, 0ull};
      // weights in place, then their high parts and remainders packed two keys to a column over the score buffer
      auto half = [&](uint32_t (&sx)[32], int col) {
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int e = 0; e < 32; e += 2) {
          float a0, a1;
          unpack_f32x2(fma_f32x2(pack_f32x2(__uint_as_float(sx[e]), __uint_as_float(sx[e + 1])), sc2, nm2), a0, a1);
          a0 = ex2_approx(a0); a1 = ex2_approx(a1);
          acc[(e >> 1) & 1] = add_f32x2(acc[(e >> 1) & 1], pack_f32x2(a0, a1));
          const uint32_t hw = pack2_t<T>(a0, a1);
          hi[e >> 1] = hw;
          const T* hv = reinterpret_cast<const T*>(&hw);
          lo[e >> 1] = pack2_t<T>(a0 - Cvt<T>::to(hv[0]), a1 - Cvt<T>::to(hv[1]));
        }
        tmem_st_32x16(tmem_s(t, sb) + lane_addr + (uint32_t)col, hi);
        tmem_st_32x16(tmem_s(t, sb) + lane_addr + (uint32_t)(32 + col), lo);
      };
      half(s0, 0);
      half(s1, 16);
      {
        float x0, x1;
        unpack_f32x2(add_f32x2(acc[0], acc[1]), x0, x1);
        l_run += x0 + x1;
      }
      tmem_st_wait();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[t][sb]);
    }
    if (ok && n_blocks > 0) {
      const int last = n_blocks - 1;
      if (__all_sync(0xffffffffu, mbar_wait(&o_full[t][last & 1], (uint32_t)((last >> 1) & 1), p.status, 40))) {
        tc_fence_after_sync();
        const float inv = 1.0f / l_run;
        T* dst = reinterpret_cast<T*>(p.y) + (long long)b * p.y_b + (long long)h * p.y_h + (long long)row * p.y_t;
        for (int c = 0; c < o_cols; c++) {
          uint32_t o[32];
          tmem_ld_32x32(tmem_o(t) + lane_addr + (uint32_t)(c * 32), o);
          tmem_ld_wait();
          if (row >= p.tq) continue;
          if (p.y_vec && c * 32 + 32 <= p.vdim) {
#pragma unroll
            for (int q = 0; q < 4; q++) {
              uint4 w;
              w.x = pack2_t<T>(__uint_as_float(o[q * 8 + 0]) * inv, __uint_as_float(o[q * 8 + 1]) * inv);
              w.y = pack2_t<T>(__uint_as_float(o[q * 8 + 2]) * inv, __uint_as_float(o[q * 8 + 3]) * inv);
              w.z = pack2_t<T>(__uint_as_float(o[q * 8 + 4]) * inv, __uint_as_float(o[q * 8 + 5]) * inv);
              w.w = pack2_t<T>(__uint_as_float(o[q * 8 + 6]) * inv, __uint_as_float(o[q * 8 + 7]) * inv);
              *reinterpret_cast<uint4*>(dst + c * 32 + q * 8) = w;
            }
          } else {
#pragma unroll
            for (int e = 0; e < 32; e++) if (c * 32 + e < p.vdim) dst[c * 32 + e] = Cvt<T>::from(__uint_as_float(o[e]) * inv);
          }
        }
        tc_fence_before_sync();
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  if (warp == 1) tmem_dealloc(tmem_base, 512);
}

static int lt_panels(int n) { return (n + kLtPanel - 1) / kLtPanel; }
static int lt_tiles(int vdim) { return vdim <= 128 ? 2 : 1; }
static int lt_stages(int nt, int qp, int pv) {
  const int left = kLtSmemMax - 1024 - nt * qp * kLtQPanel, per = (qp + pv) * kLtKPanel;
  const int s = left / per;
  return s > kLtMaxStages ? kLtMaxStages : s;
}

// 16-bit storage, sizes and addresses the tensor maps can describe, heads within tensor memory and shared memory.
bool latent_prefill_tc_eligible(const LatentPrefillDesc& d) {
  if (!(d.dtype == DType::BF16 || d.dtype == DType::F16)) return false;
  if (!(d.scale > 0.f) || d.dim < 1 || d.dim % 8 || d.rot_dim < 1 || d.rot_dim % 8 || d.vdim < 8 || d.vdim % 8 || d.vdim > 256) return false;
  const int qp = lt_panels(d.dim) + lt_panels(d.rot_dim), nt = lt_tiles(d.vdim);
  if (qp > 6 || lt_stages(nt, qp, lt_panels(d.vdim)) < 2) return false;
  if (d.q_ld % 8 || d.kv_ld % 8 || d.v_off % 8 || d.k_rot_ld % 8 || d.q_b % 8 || d.kv_b % 8 || d.k_rot_b % 8) return false;
  if (!aligned16(d.q) || !aligned16(d.kv) || !aligned16(d.k_rot)) return false;
  return (int64_t)d.n_seq * d.heads * ((d.T + kLtQ - 1) / kLtQ) < 0x3fffffff && d.T > 0 && d.past >= 0 && matmul_status_word() != nullptr;
}

template <typename T, int NT>
static cudaError_t launch_lt(cudaStream_t s, const CUtensorMap* m, const LatTcParams& p, int grid, int smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(latent_attention_tc_kernel<T, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kLtSmemMax);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  return launch_pdl(latent_attention_tc_kernel<T, NT>, dim3((unsigned)grid), dim3(64 + NT * 128), (size_t)smem, s, m[0], m[1], m[2], m[3], m[4], p);
}

Status latent_prefill_tc(cudaStream_t s, const LatentPrefillDesc& d) {
  const uint64_t T = (uint64_t)d.T, keys = (uint64_t)d.past + d.T, H = (uint64_t)d.heads, B = (uint64_t)d.n_seq;
  const uint8_t* q = static_cast<const uint8_t*>(d.q);
  const uint8_t* kv = static_cast<const uint8_t*>(d.kv);
  CUtensorMap m[5];
  AG_RETURN_IF_ERROR(make_map(&m[0], d.dtype, q, (uint64_t)d.dim, T, H, B, (uint64_t)d.q_ld, (uint64_t)(d.dim + d.rot_dim), (uint64_t)d.q_b, kLtPanel, kLtQ));
  AG_RETURN_IF_ERROR(make_map(&m[1], d.dtype, q + (size_t)d.dim * 2, (uint64_t)d.rot_dim, T, H, B, (uint64_t)d.q_ld, (uint64_t)(d.dim + d.rot_dim), (uint64_t)d.q_b, kLtPanel, kLtQ));
  AG_RETURN_IF_ERROR(make_map(&m[2], d.dtype, kv, (uint64_t)d.dim, keys, H, B, (uint64_t)d.kv_ld, (uint64_t)d.dim, (uint64_t)d.kv_b, kLtPanel, kLtKeys));
  AG_RETURN_IF_ERROR(make_map(&m[3], d.dtype, d.k_rot, (uint64_t)d.rot_dim, keys, 1, B, (uint64_t)d.k_rot_ld, 0, (uint64_t)d.k_rot_b, kLtPanel, kLtKeys));
  AG_RETURN_IF_ERROR(make_map(&m[4], d.dtype, kv + (size_t)d.v_off * 2, (uint64_t)d.vdim, keys, H, B, (uint64_t)d.kv_ld, (uint64_t)d.vdim, (uint64_t)d.kv_b, kLtPanel, kLtKeys));
  LatTcParams p;
  p.y = d.y; p.y_b = d.y_b; p.y_h = d.vdim; p.y_t = d.y_ld; p.heads = d.heads; p.bh = d.n_seq * d.heads; p.tq = d.T; p.past = d.past;
  p.dim = d.dim; p.rot = d.rot_dim; p.vdim = d.vdim; p.pd = lt_panels(d.dim); p.pr = lt_panels(d.rot_dim); p.pv = lt_panels(d.vdim);
  const int nt = lt_tiles(d.vdim), qp = p.pd + p.pr;
  p.stages = lt_stages(nt, qp, p.pv);
  p.pairs = (d.T + nt * kLtQ - 1) / (nt * kLtQ);
  p.y_vec = aligned16(d.y) && d.y_ld % 8 == 0 && d.y_b % 8 == 0 ? 1 : 0;
  p.scale_log2 = d.scale * 1.4426950408889634f;
  p.status = matmul_status_word();
  const int smem = nt * qp * kLtQPanel + p.stages * (qp + p.pv) * kLtKPanel + 1024, grid = p.pairs * p.bh;
  cudaError_t e;
  if (d.dtype == DType::BF16) e = nt == 2 ? launch_lt<__nv_bfloat16, 2>(s, m, p, grid, smem) : launch_lt<__nv_bfloat16, 1>(s, m, p, grid, smem);
  else e = nt == 2 ? launch_lt<__half, 2>(s, m, p, grid, smem) : launch_lt<__half, 1>(s, m, p, grid, smem);
  return cuda_status(e, "latent prefill (tcgen05)");
}

}}  // namespace ag::k
