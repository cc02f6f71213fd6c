// Prompt attention on tcgen05: query / key rows of up to 384 entries made of a part per head (or per group of heads) and,
// for the latent kind, a part whose keys all heads share; values of up to 256, keys behind any number of cached tokens. Windows
// and capped scores are a variant of their own (GEN): blocks in front of a tile pair's first window are not loaded.
//
// Built like attention_tc.cu, for wider heads. A CTA takes NT = 2 neighbouring tiles of 128 query rows of one head (NT = 1
// above 128 value columns) and walks their keys in blocks of 64, every K and V block loaded once for both tiles: warp 0
// loads (TMA, 64-column panels: the heads' own part, zero-filled past its end, then the shared one, each from its own
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

constexpr int kPtQ = 128, kPtKeys = 64, kPtPanel = 64, kPtMaxStages = 4;
constexpr int kPtQPanel = kPtQ * kPtPanel * 2, kPtKPanel = kPtKeys * kPtPanel * 2;
constexpr int kPtSmemMax = 226 * 1024;
constexpr float kPtRescaleLog2 = 8.0f;      // see attention_tc.cu: growth of the maximum that is carried without rescaling

struct PromptTcParams {
  void* y;
  long long y_b, y_h, y_t;
  int heads, group, bh, tq, past, pairs;    // group: heads per key head; pairs: query tile groups per head
  int window;                               // keys a row sees, 0: all
  int dim, rot, vdim, pd, pr, pv, stages;   // panels of the unrotated, rotated and value columns
  int y_vec;
  float scale_log2;                         // with a cap: scale / cap, and the cap in log2 units
  float cap_log2;
  int* status;
};

// 16-wide MMA steps that panel `c` of a part of `n` columns needs
__device__ __forceinline__ int pt_steps(int n, int c) { const int left = n - c * kPtPanel; return left >= kPtPanel ? 4 : (left + 15) / 16; }

// cap * tanh(x) with the hardware exp2 and reciprocal: absolute error about 2^-22 of the cap
__device__ __forceinline__ float pt_cap(float x, float cap) { return cap - __fdividef(2.0f * cap, ex2_approx(x * 2.885390081777927f) + 1.0f); }

template <typename T, int NT, bool GEN>
__global__ void __launch_bounds__(64 + NT * 128, 1)
prompt_attention_tc_kernel(const __grid_constant__ CUtensorMap mq, const __grid_constant__ CUtensorMap mqr, const __grid_constant__ CUtensorMap mk,
                           const __grid_constant__ CUtensorMap mkr, const __grid_constant__ CUtensorMap mv, const PromptTcParams p) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t q_full[NT], k_full[kPtMaxStages], k_empty[kPtMaxStages], v_full[kPtMaxStages], v_empty[kPtMaxStages], s_full[NT][2], p_full[NT][2], o_full[NT][2];
  __shared__ uint32_t tmem_base_slot;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int qp = p.pd + p.pr;
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + NT * qp * kPtQPanel;
  uint8_t* sV = sK + p.stages * qp * kPtKPanel;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < kPtMaxStages; s++) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1); }
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
  auto tmem_s = [&](int t, int b) { return tmem_base + (uint32_t)((t * 2 + b) * kPtKeys); };
  auto tmem_o = [&](int t) { return tmem_base + (uint32_t)(NT * 2 * kPtKeys + t * 128); };
  pdl_wait();
  pdl_trigger();

  // longest tiles first
  const int g = (int)blockIdx.x / p.bh, bh = (int)blockIdx.x % p.bh;
  const int b = bh / p.heads, h = bh % p.heads;
  const int q0 = (p.pairs - 1 - g) * NT * kPtQ;
  const int tk = p.past + p.tq;
  const int kh = h / p.group;
  const int base = GEN && p.window ? max(0, p.past + q0 - p.window + 1) / kPtKeys * kPtKeys : 0;      // first key of the first block
  int nb[NT], n_max = 0;
#pragma unroll
  for (int t = 0; t < NT; t++) {
    const int first = q0 + t * kPtQ;
    nb[t] = first < p.tq ? (min(tk, p.past + first + kPtQ) - base + kPtKeys - 1) / kPtKeys : 0;
    n_max = max(n_max, nb[t]);
  }

  if (warp == 0) {
    if (lane == 0) {
      bool ok = true;
      for (int t = 0; t < NT; t++) {
        if (nb[t] == 0) continue;
        mbar_expect_tx(&q_full[t], (uint32_t)(qp * kPtQPanel));
        uint8_t* dst = sQ + t * qp * kPtQPanel;
        for (int c = 0; c < p.pd; c++) tma_load_4d(dst + c * kPtQPanel, &mq, &q_full[t], c * kPtPanel, q0 + t * kPtQ, h, b);
        for (int c = 0; c < p.pr; c++) tma_load_4d(dst + (p.pd + c) * kPtQPanel, &mqr, &q_full[t], c * kPtPanel, q0 + t * kPtQ, h, b);
      }
      for (int j = 0; j < n_max && ok; j++) {
        const int st = j % p.stages;
        const uint32_t ph = (uint32_t)((j / p.stages) & 1);
        if (!mbar_wait(&k_empty[st], ph ^ 1, p.status, 32)) { ok = false; break; }
        mbar_expect_tx(&k_full[st], (uint32_t)(qp * kPtKPanel));
        uint8_t* dk = sK + st * qp * kPtKPanel;
        for (int c = 0; c < p.pd; c++) tma_load_4d(dk + c * kPtKPanel, &mk, &k_full[st], c * kPtPanel, base + j * kPtKeys, kh, b);
        for (int c = 0; c < p.pr; c++) tma_load_4d(dk + (p.pd + c) * kPtKPanel, &mkr, &k_full[st], c * kPtPanel, base + j * kPtKeys, 0, b);
        if (!mbar_wait(&v_empty[st], ph ^ 1, p.status, 33)) { ok = false; break; }
        mbar_expect_tx(&v_full[st], (uint32_t)(p.pv * kPtKPanel));
        uint8_t* dv = sV + st * p.pv * kPtKPanel;
        for (int c = 0; c < p.pv; c++) tma_load_4d(dv + c * kPtKPanel, &mv, &v_full[st], c * kPtPanel, base + j * kPtKeys, kh, b);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr int fmt = std::is_same<T, __nv_bfloat16>::value ? 1 : 0;
      const uint32_t idesc_s = make_idesc_f16(fmt, 0, 0, kPtQ, kPtKeys);
      const uint32_t idesc_o = make_idesc_f16(fmt, 0, 1, kPtQ, (p.vdim + 15) / 16 * 16);
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
            const uint32_t a = smem_u32(sQ + (t * qp + c) * kPtQPanel), bb = smem_u32(sK + (st * qp + c) * kPtKPanel);
            const int steps = c < p.pd ? pt_steps(p.dim, c) : pt_steps(p.rot, c - p.pd);
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
          const uint32_t bb = smem_u32(sV + st * p.pv * kPtKPanel);
#pragma unroll
          for (int part = 0; part < 2; part++)
#pragma unroll
            for (int kk = 0; kk < kPtKeys / 16; kk++)
              mma_f16_ts(tmem_o(t), tmem_s(t, j & 1) + (uint32_t)(part * 32 + kk * 8), make_smem_desc_sw128(bb + kk * 2048, kPtKPanel, 1024), idesc_o,
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
    const int row = q0 + t * kPtQ + r;
    const float sc = GEN && p.cap_log2 > 0.f ? 1.0f : p.scale_log2;
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
      if constexpr (GEN) {
        if (p.cap_log2 > 0.f) {
#pragma unroll
          for (int e = 0; e < 32; e++) {
            s0[e] = __float_as_uint(pt_cap(__uint_as_float(s0[e]) * p.scale_log2, p.cap_log2));
            s1[e] = __float_as_uint(pt_cap(__uint_as_float(s1[e]) * p.scale_log2, p.cap_log2));
          }
        }
        const int low = p.window ? p.past + row - p.window + 1 - base - j * kPtKeys : 0;      // first column inside the row's window
        if (__any_sync(0xffffffffu, low > 0)) {
#pragma unroll
          for (int e = 0; e < 32; e++) {
            if (e < low) s0[e] = 0xff800000u;
            if (32 + e < low) s1[e] = 0xff800000u;
          }
        }
      }
      const int lim = min(min(tk, p.past + row + 1) - base - j * kPtKeys, kPtKeys);      // columns of the block this row sees
      if (!__all_sync(0xffffffffu, lim >= kPtKeys)) {
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
      const bool moves = (m_cand - m_ref > kPtRescaleLog2) || (m_ref == -INFINITY && m_cand != -INFINITY);
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

static int pt_panels(int n) { return (n + kPtPanel - 1) / kPtPanel; }
static int pt_tiles(int vdim) { return vdim <= 128 ? 2 : 1; }
static int pt_stages(int nt, int qp, int pv) {
  const int left = kPtSmemMax - 1024 - nt * qp * kPtQPanel, per = (qp + pv) * kPtKPanel;
  const int s = left / per;
  return s > kPtMaxStages ? kPtMaxStages : s;
}

// 16-bit storage, sizes and addresses the tensor maps can describe, heads within tensor memory and shared memory.
bool prompt_attention_tc_eligible(const PromptAttnDesc& d) {
  if (!(d.dtype == DType::BF16 || d.dtype == DType::F16)) return false;
  if (!(d.scale > 0.f) || d.dim < 1 || d.dim % 8 || d.rot_dim < 0 || d.rot_dim % 8 || d.vdim < 8 || d.vdim % 8 || d.vdim > 256) return false;
  const int qp = pt_panels(d.dim) + pt_panels(d.rot_dim), nt = pt_tiles(d.vdim);
  if (qp > 6 || pt_stages(nt, qp, pt_panels(d.vdim)) < 2) return false;
  if (d.q_ld % 8 || d.k_ld % 8 || d.v_ld % 8 || d.k_rot_ld % 8 || d.q_b % 8 || d.k_b % 8 || d.v_b % 8 || d.k_rot_b % 8) return false;
  if (!aligned16(d.q) || !aligned16(d.k) || !aligned16(d.v) || !aligned16(d.k_rot)) return false;
  return (int64_t)d.n_seq * d.heads * ((d.T + kPtQ - 1) / kPtQ) < 0x3fffffff && d.T > 0 && d.past >= 0 && matmul_status_word() != nullptr;
}

template <typename T, int NT, bool GEN>
static cudaError_t launch_pt(cudaStream_t s, const CUtensorMap* m, const PromptTcParams& p, int grid, int smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(prompt_attention_tc_kernel<T, NT, GEN>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPtSmemMax);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  return launch_pdl(prompt_attention_tc_kernel<T, NT, GEN>, dim3((unsigned)grid), dim3(64 + NT * 128), (size_t)smem, s, m[0], m[1], m[2], m[3], m[4], p);
}

Status prompt_attention_tc(cudaStream_t s, const PromptAttnDesc& d) {
  const uint64_t T = (uint64_t)d.T, keys = (uint64_t)d.past + d.T, H = (uint64_t)d.heads, B = (uint64_t)d.n_seq;
  const uint8_t* q = static_cast<const uint8_t*>(d.q);
  const uint64_t G = H / (uint64_t)d.group;
  CUtensorMap m[5];
  AG_RETURN_IF_ERROR(make_map(&m[0], d.dtype, q, (uint64_t)d.dim, T, H, B, (uint64_t)d.q_ld, (uint64_t)(d.dim + d.rot_dim), (uint64_t)d.q_b, kPtPanel, kPtQ));
  AG_RETURN_IF_ERROR(make_map(&m[2], d.dtype, d.k, (uint64_t)d.dim, keys, G, B, (uint64_t)d.k_ld, (uint64_t)d.dim, (uint64_t)d.k_b, kPtPanel, kPtKeys));
  if (d.rot_dim) {
    AG_RETURN_IF_ERROR(make_map(&m[1], d.dtype, q + (size_t)d.dim * 2, (uint64_t)d.rot_dim, T, H, B, (uint64_t)d.q_ld, (uint64_t)(d.dim + d.rot_dim), (uint64_t)d.q_b, kPtPanel, kPtQ));
    AG_RETURN_IF_ERROR(make_map(&m[3], d.dtype, d.k_rot, (uint64_t)d.rot_dim, keys, 1, B, (uint64_t)d.k_rot_ld, 0, (uint64_t)d.k_rot_b, kPtPanel, kPtKeys));
  } else { m[1] = m[0]; m[3] = m[2]; }               // no shared part: never loaded
  AG_RETURN_IF_ERROR(make_map(&m[4], d.dtype, d.v, (uint64_t)d.vdim, keys, G, B, (uint64_t)d.v_ld, (uint64_t)d.vdim, (uint64_t)d.v_b, kPtPanel, kPtKeys));
  PromptTcParams p;
  p.y = d.y; p.y_b = d.y_b; p.y_h = d.vdim; p.y_t = d.y_ld; p.heads = d.heads; p.group = d.group; p.window = d.window; p.bh = d.n_seq * d.heads; p.tq = d.T; p.past = d.past;
  p.dim = d.dim; p.rot = d.rot_dim; p.vdim = d.vdim; p.pd = pt_panels(d.dim); p.pr = pt_panels(d.rot_dim); p.pv = pt_panels(d.vdim);
  const int nt = pt_tiles(d.vdim), qp = p.pd + p.pr;
  p.stages = pt_stages(nt, qp, p.pv);
  p.pairs = (d.T + nt * kPtQ - 1) / (nt * kPtQ);
  p.y_vec = aligned16(d.y) && d.y_ld % 8 == 0 && d.y_b % 8 == 0 ? 1 : 0;
  const bool cap = d.softcap > 0.f, gen = cap || d.window;
  p.scale_log2 = cap ? d.scale / d.softcap : d.scale * 1.4426950408889634f;
  p.cap_log2 = cap ? d.softcap * 1.4426950408889634f : 0.f;
  p.status = matmul_status_word();
  const int smem = nt * qp * kPtQPanel + p.stages * (qp + p.pv) * kPtKPanel + 1024, grid = p.pairs * p.bh;
  cudaError_t e;
  auto launch = [&](auto tag) {
    using T = decltype(tag);
    if (nt == 2) return gen ? launch_pt<T, 2, true>(s, m, p, grid, smem) : launch_pt<T, 2, false>(s, m, p, grid, smem);
    return gen ? launch_pt<T, 1, true>(s, m, p, grid, smem) : launch_pt<T, 1, false>(s, m, p, grid, smem);
  };
  if (d.dtype == DType::BF16) e = launch(__nv_bfloat16()); else e = launch(__half());
  return cuda_status(e, "prompt attention (tcgen05)");
}

}}  // namespace ag::k
