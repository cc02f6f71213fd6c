// The two heavy steps of an mLSTM portion on tcgen05: what each chunk adds to the state, and the chunk's outputs.
//
// Factors that the recurrence wants in float32 (decayed keys, the state, decayed scores) enter the products as the sum of
// two 16-bit numbers, a high part and its remainder, so a product rounds them at 2^-16 or below instead of at the storage
// type's step; queries, keys and values are storage-type values to begin with. All waits are bounded.
#include "mlstm.cuh"
#include "sm100.cuh"
#include "tc_math.cuh"
#include <cuda.h>
#include <type_traits>

namespace ag { namespace k {

using namespace ag::sm100;

Status make_map(CUtensorMap* out, DType dt, const void* ptr, uint64_t inner, uint64_t rows, uint64_t nbi, uint64_t nbo,
                uint64_t row_stride, uint64_t bi_stride, uint64_t bo_stride, uint32_t b0, uint32_t b1);

constexpr int kMtPanel = 64, kMtTok = 64;                      // columns per TMA panel, tokens per block
constexpr int kMtPanelBytes = kMtTok * kMtPanel * 2;           // 8 KB
constexpr int kMtSmemMax = 226 * 1024;

__device__ __forceinline__ float ml_pow(float4 row, float4 key, float m2) { return ex2_approx((row.x + key.z) + ((row.y + key.w) - m2)); }

// ── chunk: U = sum_j w_j k_j v_j^T and n = sum_j w_j k_j over the chunk's tokens ────────────────────────────────
// D[dim, vdim] = A[dim, tokens] B[tokens, vdim], both operands as they lie (tokens are rows, so A is M-major and B N-major).
// Four converter warps scale the key rows by their decay in shared memory and split them; they also hold the sum for n and
// write the result. grid: (chunks x tiles of 128 key dimensions x tiles of 256 value columns, n_seq * heads).
constexpr int kMcStages = 3;
struct MlChunkTc { MlParams p; int m_tiles, n_tiles, pv; int* status; };
template <typename T>
__global__ void __launch_bounds__(192, 1) ml_chunk_tc_kernel(const __grid_constant__ CUtensorMap mk, const __grid_constant__ CUtensorMap mv, const MlChunkTc a) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t k_full[kMcStages], v_full[kMcStages], c_full[kMcStages], empty[kMcStages], acc_full;
  __shared__ uint32_t tmem_base_slot;
  __shared__ float s_n[8][128];
  __shared__ float s_w[kMlChunk];
  const MlParams& p = a.p;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int stage_bytes = (4 + a.pv) * kMtPanelBytes;          // keys: high part (2 panels), remainder (2), values
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < kMcStages; s++) { mbar_init(&k_full[s], 1); mbar_init(&v_full[s], 1); mbar_init(&c_full[s], 4); mbar_init(&empty[s], 1); }
    mbar_init(&acc_full, 1);
    mbar_fence_init();
    prefetch_tmap(&mk); prefetch_tmap(&mv);
  }
  if (warp == 1) { tmem_alloc(&tmem_base_slot, 256); tmem_relinquish(); }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = tmem_base_slot;
  pdl_wait();
  pdl_trigger();
  const int e0 = (int)blockIdx.x % a.n_tiles * 256, d0 = (int)blockIdx.x / a.n_tiles % a.m_tiles * 128, c = (int)blockIdx.x / (a.n_tiles * a.m_tiles);
  const int ne = min(256, p.vdim - e0);
  const int sh = blockIdx.y, s = sh / p.heads, h = sh % p.heads;
  const int t0 = c * kMlChunk, t1 = min(p.T, t0 + kMlChunk), blocks = (t1 - t0 + kMtTok - 1) / kMtTok;
  if (warp == 0) {
    if (lane == 0) {
      for (int j = 0; j < blocks; j++) {
        const int st = j % kMcStages;
        if (!mbar_wait(&empty[st], (uint32_t)((j / kMcStages) & 1) ^ 1, a.status, 44)) break;
        uint8_t* base = smem + st * stage_bytes;
        mbar_expect_tx(&k_full[st], 2 * kMtPanelBytes);
        for (int q = 0; q < 2; q++) tma_load_4d(base + q * kMtPanelBytes, &mk, &k_full[st], d0 + q * kMtPanel, t0 + j * kMtTok, h, s);
        mbar_expect_tx(&v_full[st], (uint32_t)(a.pv * kMtPanelBytes));
        for (int q = 0; q < a.pv; q++) tma_load_4d(base + (4 + q) * kMtPanelBytes, &mv, &v_full[st], e0 + q * kMtPanel, t0 + j * kMtTok, h, s);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr int fmt = std::is_same<T, __nv_bfloat16>::value ? 1 : 0;
      const uint32_t idesc = make_idesc_f16(fmt, 1, 1, 128, (ne + 15) / 16 * 16);
      bool ok = true;
      for (int j = 0; j < blocks && ok; j++) {
        const int st = j % kMcStages;
        const uint32_t ph = (uint32_t)((j / kMcStages) & 1);
        ok = mbar_wait(&c_full[st], ph, a.status, 45) && mbar_wait(&v_full[st], ph, a.status, 46);
        if (!ok) break;
        tc_fence_after_sync();
        const uint32_t base = smem_u32(smem + st * stage_bytes), bb = base + 4 * kMtPanelBytes;
#pragma unroll
        for (int part = 0; part < 2; part++)
#pragma unroll
          for (int kk = 0; kk < kMtTok / 16; kk++)
            mma_f16_ss(tmem, make_smem_desc_sw128(base + part * 2 * kMtPanelBytes + kk * 2048, kMtPanelBytes, 1024), make_smem_desc_sw128(bb + kk * 2048, kMtPanelBytes, 1024),
                       idesc, (j > 0 || part > 0 || kk > 0) ? 1u : 0u);
        mma_commit(&empty[st]);
      }
      if (ok) mma_commit(&acc_full);
    }
  } else {
    const int tid = threadIdx.x - 64;
    const float4* ab = p.w.ab + (long long)sh * p.T;
    const float4 end = ab[t1 - 1];
    const float m_end = p.w.m2[(long long)sh * p.T + t1 - 1];
    for (int i = tid; i < kMlChunk; i += 128) s_w[i] = t0 + i < t1 ? ml_pow(end, ab[t0 + i], m_end) : 0.f;
    asm volatile("bar.sync 1, 128;" ::: "memory");
    const int ch = tid & 15, r0 = tid >> 4;                    // a 16-byte piece of the 128 columns, rows r0, r0 + 8, ...
    float nacc[8];
#pragma unroll
    for (int e = 0; e < 8; e++) nacc[e] = 0.f;
    bool ok = true;
    for (int j = 0; j < blocks; j++) {
      const int st = j % kMcStages;
      if (!__all_sync(0xffffffffu, mbar_wait(&k_full[st], (uint32_t)((j / kMcStages) & 1), a.status, 47))) { ok = false; break; }
      uint8_t* base = smem + st * stage_bytes + (ch >> 3) * kMtPanelBytes;
#pragma unroll
      for (int i = 0; i < 8; i++) {
        const int row = r0 + 8 * i;
        const float w = s_w[j * kMtTok + row];
        uint8_t* at = base + row * 128 + (((ch & 7) ^ (row & 7)) << 4);
        const uint4 raw = *reinterpret_cast<const uint4*>(at);
        const T* v = reinterpret_cast<const T*>(&raw);
        uint4 hi, lo;
        uint32_t* hp = reinterpret_cast<uint32_t*>(&hi);
        uint32_t* lp = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
        for (int e = 0; e < 4; e++) {
          const float x0 = Cvt<T>::to(v[2 * e]) * w, x1 = Cvt<T>::to(v[2 * e + 1]) * w;
          nacc[2 * e] += x0; nacc[2 * e + 1] += x1;
          hp[e] = pack2_t<T>(x0, x1);
          const T* hv = reinterpret_cast<const T*>(&hp[e]);
          lp[e] = pack2_t<T>(x0 - Cvt<T>::to(hv[0]), x1 - Cvt<T>::to(hv[1]));
        }
        *reinterpret_cast<uint4*>(at) = hi;
        *reinterpret_cast<uint4*>(at + 2 * kMtPanelBytes) = lo;
      }
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(&c_full[st]);
    }
#pragma unroll
    for (int e = 0; e < 8; e++) s_n[r0][ch * 8 + e] = nacc[e];
    asm volatile("bar.sync 1, 128;" ::: "memory");
    const long long ci = (long long)sh * p.w.chunks + c;
    if (e0 == 0 && d0 + tid < p.dim) {
      float v = 0.f;
#pragma unroll
      for (int r = 0; r < 8; r++) v += s_n[r][tid];
      p.w.n[ci * p.dim + d0 + tid] = v;
    }
    if (ok && __all_sync(0xffffffffu, mbar_wait(&acc_full, 0, a.status, 48))) {
      tc_fence_after_sync();
      const int quarter = warp & 3, row = d0 + quarter * 32 + lane;
      float* dst = p.w.S + (ci * p.dim + row) * p.vdim + e0;
      for (int g = 0; g * 32 < ne; g++) {
        uint32_t o[32];
        tmem_ld_32x32(tmem + ((uint32_t)(quarter * 32) << 16) + (uint32_t)(g * 32), o);
        tmem_ld_wait();
        if (row >= p.dim) continue;
#pragma unroll
        for (int q = 0; q < 8; q++)
          if (g * 32 + q * 4 < ne) *reinterpret_cast<uint4*>(dst + g * 32 + q * 4) = make_uint4(o[q * 4], o[q * 4 + 1], o[q * 4 + 2], o[q * 4 + 3]);
      }
      tc_fence_before_sync();
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  if (warp == 1) tmem_dealloc(tmem, 256);
}

// ── output ──────────────────────────────────────────────────────────────────
// A cluster: 128 rows of one head, each CTA 128 value columns (the scores are computed by every one; the head norm's sums meet
// over distributed shared memory), small enough for two CTAs per SM. O = (q S) r first (the state's planes stream through the value ring), then the chunk's key
// blocks: scores by tcgen05, times their decay by the row's thread, split, O += P V from tensor memory. The row's thread
// also holds n . q, so it ends with the division, the head norm, the norm weight and the output gate.
constexpr int kMoCols = 128;
struct MlOutTc { MlParams p; int pd, pv, ks, vs, ranks, y_vec; int* status; };
constexpr int kMoMaxStages = 4;
template <typename T>
__global__ void __launch_bounds__(192, 2) ml_output_tc_kernel(const __grid_constant__ CUtensorMap mq, const __grid_constant__ CUtensorMap mk, const __grid_constant__ CUtensorMap mv,
                                                           const __grid_constant__ CUtensorMap ms, const MlOutTc a) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t q_full, k_full[kMoMaxStages], k_empty[kMoMaxStages], v_full[kMoMaxStages], v_empty[kMoMaxStages], s_full[2], p_full[2], st_full, st_done, o_full;
  __shared__ uint32_t tmem_base_slot;
  __shared__ __align__(16) float2 s_b[kMlChunk];
  __shared__ float s_n[256];
  __shared__ float s_sq[128];
  const MlParams& p = a.p;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* sQ = smem;                                          // pd panels of 128 rows
  uint8_t* sK = sQ + a.pd * 2 * kMtPanelBytes;                 // ks stages of pd panels
  uint8_t* sV = sK + a.ks * a.pd * kMtPanelBytes;              // vs stages of pv panels
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(&q_full, 1); mbar_init(&st_full, 1); mbar_init(&st_done, 4); mbar_init(&o_full, 1);
    for (int s = 0; s < kMoMaxStages; s++) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1); }
    for (int s = 0; s < 2; s++) { mbar_init(&s_full[s], 1); mbar_init(&p_full[s], 4); }
    mbar_fence_init();
    prefetch_tmap(&mq); prefetch_tmap(&mk); prefetch_tmap(&mv); prefetch_tmap(&ms);
  }
  if (warp == 1) { tmem_alloc(&tmem_base_slot, 256); tmem_relinquish(); }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_s = tmem_base_slot, tmem_o = tmem_base_slot + 2 * kMtTok;
  pdl_wait();
  pdl_trigger();
  const int rank = (int)blockIdx.x % a.ranks, e0 = rank * kMoCols, ne = min(kMoCols, p.vdim - e0);
  const int q0 = (int)((gridDim.x - 1 - blockIdx.x) / a.ranks) * 128, sh = blockIdx.y, s = sh / p.heads, h = sh % p.heads;
  const int c = q0 / kMlChunk, t0 = c * kMlChunk;
  const int blocks = (min(p.T, q0 + 128) - t0 + kMtTok - 1) / kMtTok;
  const int dblocks = (p.dim + kMtTok - 1) / kMtTok, vblocks = 2 * dblocks;       // state planes in blocks of 64 rows, ahead of the values
  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(&q_full, (uint32_t)(a.pd * 2 * kMtPanelBytes));
      for (int q = 0; q < a.pd; q++) tma_load_4d(sQ + q * 2 * kMtPanelBytes, &mq, &q_full, q * kMtPanel, q0, h, s);
      bool ok = true;
      int jk = 0, jv = 0;
      auto load_k = [&]() {
        const int st = jk % a.ks;
        if (!mbar_wait(&k_empty[st], (uint32_t)((jk / a.ks) & 1) ^ 1, a.status, 50)) { ok = false; return; }
        mbar_expect_tx(&k_full[st], (uint32_t)(a.pd * kMtPanelBytes));
        for (int q = 0; q < a.pd; q++) tma_load_4d(sK + (st * a.pd + q) * kMtPanelBytes, &mk, &k_full[st], q * kMtPanel, t0 + jk * kMtTok, h, s);
        jk++;
      };
      auto load_v = [&]() {
        const int st = jv % a.vs;
        if (!mbar_wait(&v_empty[st], (uint32_t)((jv / a.vs) & 1) ^ 1, a.status, 51)) { ok = false; return; }
        mbar_expect_tx(&v_full[st], (uint32_t)(a.pv * kMtPanelBytes));
        uint8_t* dst = sV + st * a.pv * kMtPanelBytes;
        for (int q = 0; q < a.pv; q++) {
          if (jv < vblocks) tma_load_4d(dst + q * kMtPanelBytes, &ms, &v_full[st], e0 + q * kMtPanel, (jv >> 1) * kMtTok, c * 2 + (jv & 1), sh);
          else tma_load_4d(dst + q * kMtPanelBytes, &mv, &v_full[st], e0 + q * kMtPanel, t0 + (jv - vblocks) * kMtTok, h, s);
        }
        jv++;
      };
      load_k();
      if (ok && blocks > 1) load_k();
      while (ok && jv < vblocks) load_v();
      while (ok && jv < vblocks + blocks) {
        load_v();
        if (ok && jk < blocks) load_k();
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr int fmt = std::is_same<T, __nv_bfloat16>::value ? 1 : 0;
      const uint32_t idesc_s = make_idesc_f16(fmt, 0, 0, 128, kMtTok), idesc_o = make_idesc_f16(fmt, 0, 1, 128, (ne + 15) / 16 * 16);
      auto steps = [&](int q) { const int left = p.dim - q * kMtPanel; return left >= kMtPanel ? 4 : (left + 15) / 16; };
      auto issue_s = [&](int j) -> bool {
        if (j >= blocks) return true;
        const int st = j % a.ks;
        if (!mbar_wait(&k_full[st], (uint32_t)((j / a.ks) & 1), a.status, 52)) return false;
        tc_fence_after_sync();
        uint32_t acc = 0;
        for (int q = 0; q < a.pd; q++) {
          const uint32_t x = smem_u32(sQ + q * 2 * kMtPanelBytes), y = smem_u32(sK + (st * a.pd + q) * kMtPanelBytes);
          for (int kk = 0; kk < steps(q); kk++, acc = 1)
            mma_f16_ss(tmem_s + (uint32_t)((j & 1) * kMtTok), make_smem_desc_sw128(x + kk * 32, 16, 1024), make_smem_desc_sw128(y + kk * 32, 16, 1024), idesc_s, acc);
        }
        mma_commit(&k_empty[st]);
        mma_commit(&s_full[j & 1]);
        return true;
      };
      bool ok = mbar_wait(&q_full, 0, a.status, 53);
      if (ok) ok = issue_s(0) && issue_s(1);
      uint32_t acc = 0;
      for (int j = 0; j < vblocks && ok; j++) {
        const int st = j % a.vs, q = j >> 1;
        ok = mbar_wait(&v_full[st], (uint32_t)((j / a.vs) & 1), a.status, 54);
        if (!ok) break;
        tc_fence_after_sync();
        const uint32_t x = smem_u32(sQ + q * 2 * kMtPanelBytes), y = smem_u32(sV + st * a.pv * kMtPanelBytes);
        for (int kk = 0; kk < steps(q); kk++, acc = 1)
          mma_f16_ss(tmem_o, make_smem_desc_sw128(x + kk * 32, 16, 1024), make_smem_desc_sw128(y + kk * 2048, kMtPanelBytes, 1024), idesc_o, acc);
        mma_commit(&v_empty[st]);
      }
      if (ok) { mma_commit(&st_full); ok = mbar_wait(&st_done, 0, a.status, 55); }
      for (int j = 0; j < blocks && ok; j++) {
        const int jv = vblocks + j, st = jv % a.vs;
        ok = mbar_wait(&v_full[st], (uint32_t)((jv / a.vs) & 1), a.status, 56) && mbar_wait(&p_full[j & 1], (uint32_t)((j >> 1) & 1), a.status, 57);
        if (!ok) break;
        tc_fence_after_sync();
        const uint32_t y = smem_u32(sV + st * a.pv * kMtPanelBytes);
#pragma unroll
        for (int part = 0; part < 2; part++)
#pragma unroll
          for (int kk = 0; kk < kMtTok / 16; kk++)
            mma_f16_ts(tmem_o, tmem_s + (uint32_t)((j & 1) * kMtTok + part * 32 + kk * 8), make_smem_desc_sw128(y + kk * 2048, kMtPanelBytes, 1024), idesc_o, 1u);
        mma_commit(&v_empty[st]);
        ok = issue_s(j + 2);
      }
      if (ok) mma_commit(&o_full);
    }
  }
  // the row's thread (warps 2 .. 5)
  const int tid = threadIdx.x - 64, quarter = warp & 3, lr = quarter * 32 + lane;
  const int row = q0 + lr, rr = min(row, p.T - 1);
  const uint32_t lane_addr = (uint32_t)(quarter * 32) << 16;
  const T* grow = reinterpret_cast<const T*>(p.proj) + ((long long)s * p.T + rr) * p.ld;
  const int o_groups = (ne + 31) / 32;
  float den = 0.f;
  bool ok = warp >= 2;
  uint4 z[kMoCols / 8];
  if (warp >= 2) {
    const float4* ab = p.w.ab + (long long)sh * p.T;
    const float4 mine = ab[rr];
    const float m2 = p.w.m2[(long long)sh * p.T + rr];
    for (int i = tid; i < blocks * kMtTok; i += 128) {
      float2 b = make_float2(0.f, 0.f);
      if (t0 + i < p.T) { const float4 k = ab[t0 + i]; b = make_float2(k.z, k.w); }
      s_b[i] = b;
    }
    const float* n = p.w.n + ((long long)sh * p.w.chunks + c) * p.dim;
    for (int i = tid; i < p.dim; i += 128) s_n[i] = n[i];
    asm volatile("bar.sync 1, 128;" ::: "memory");
    // what lies in front of the chunk reaches this row by r
    const float m_c = p.w.m_start[(long long)sh * (p.w.chunks + 1) + c] * 1.4426950408889634f;
    const float r = ex2_approx((mine.x + m_c) + (mine.y - m2)) * p.q_scale;
    float nq = 0.f;
    ok = __all_sync(0xffffffffu, mbar_wait(&q_full, 0, a.status, 49));
    if (ok) {
      for (int i = 0; i < p.dim; i += 8) {
        const uint4 raw = *reinterpret_cast<const uint4*>(sQ + (i >> 6) * 2 * kMtPanelBytes + lr * 128 + ((((i & 63) >> 3) ^ (lr & 7)) << 4));
        const T* v = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int e = 0; e < 8; e++) nq = fmaf(Cvt<T>::to(v[e]), s_n[i + e], nq);
      }
      nq *= r;
    }
    ok = ok && __all_sync(0xffffffffu, mbar_wait(&st_full, 0, a.status, 58));
    if (ok) {
      tc_fence_after_sync();
      for (int g = 0; g < o_groups; g++) {
        uint32_t o[32];
        tmem_ld_32x32(tmem_o + lane_addr + (uint32_t)(g * 32), o);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 32; e++) o[e] = __float_as_uint(__uint_as_float(o[e]) * r);
        tmem_st_32x32(tmem_o + lane_addr + (uint32_t)(g * 32), o);
      }
      tmem_st_wait();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&st_done);
    }
    const float row_lo = mine.y - m2;
    for (int j = 0; j < blocks && ok; j++) {
      const int sb = j & 1;
      if (!__all_sync(0xffffffffu, mbar_wait(&s_full[sb], (uint32_t)((j >> 1) & 1), a.status, 59))) { ok = false; break; }
      tc_fence_after_sync();
      const int lim = row - (t0 + j * kMtTok) + 1;             // keys of the block this row sees
      const bool full = __all_sync(0xffffffffu, lim >= kMtTok);
      uint32_t s0[32], s1[32];
      tmem_ld_32x32(tmem_s + lane_addr + (uint32_t)(sb * kMtTok), s0);
      tmem_ld_32x32(tmem_s + lane_addr + (uint32_t)(sb * kMtTok + 32), s1);
      tmem_ld_wait();
      auto half = [&](const uint32_t (&sx)[32], int col) {
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int e = 0; e < 32; e += 2) {
          const float4 b = *reinterpret_cast<const float4*>(&s_b[j * kMtTok + col + e]);        // (b, remainder) of two keys
          const float w0 = ex2_approx((mine.x + b.x) + (row_lo + b.y)), w1 = ex2_approx((mine.x + b.z) + (row_lo + b.w));
          float x0 = __uint_as_float(sx[e]) * p.q_scale * w0, x1 = __uint_as_float(sx[e + 1]) * p.q_scale * w1;
          if (!full) { if (col + e >= lim) x0 = 0.f; if (col + e + 1 >= lim) x1 = 0.f; }
          nq += x0 + x1;
          hi[e >> 1] = pack2_t<T>(x0, x1);
          const T* hv = reinterpret_cast<const T*>(&hi[e >> 1]);
          lo[e >> 1] = pack2_t<T>(x0 - Cvt<T>::to(hv[0]), x1 - Cvt<T>::to(hv[1]));
        }
        tmem_st_32x16(tmem_s + lane_addr + (uint32_t)(sb * kMtTok + col / 2), hi);
        tmem_st_32x16(tmem_s + lane_addr + (uint32_t)(sb * kMtTok + 32 + col / 2), lo);
      };
      half(s0, 0);
      half(s1, 32);
      tmem_st_wait();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[sb]);
    }
    // the output gate's values are on their way while the last product finishes
    const T* gp = grow + 2 * p.heads * p.dim + p.heads * p.vdim + h * p.vdim + e0;
#pragma unroll
    for (int q = 0; q < kMoCols / 8; q++) z[q] = q * 8 < ne ? *reinterpret_cast<const uint4*>(gp + q * 8) : make_uint4(0u, 0u, 0u, 0u);
    ok = ok && __all_sync(0xffffffffu, mbar_wait(&o_full, 0, a.status, 60));
    if (ok) {
      tc_fence_after_sync();
      den = 1.0f / (fmaxf(fabsf(nq), ex2_approx(-m2)) + 1e-6f);
      float sq = 0.f;
      for (int g = 0; g < o_groups; g++) {
        uint32_t o[32];
        tmem_ld_32x32(tmem_o + lane_addr + (uint32_t)(g * 32), o);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 32; e++) {
          const float v = g * 32 + e < ne ? __uint_as_float(o[e]) * den : 0.f;
          sq = fmaf(v, v, sq);
        }
      }
      s_sq[lr] = sq;
    }
  }
  __syncwarp();
  if (a.ranks > 1) cluster_sync_all();
  if (ok) {
    float sq = 0.f;
    for (int q = 0; q < a.ranks; q++) {
      float v = s_sq[lr];
      if (a.ranks > 1) asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(mapa_u32(smem_u32(&s_sq[lr]), (uint32_t)q)));
      sq += v;
    }
    const float rs = den / sqrtf(sq / (float)p.vdim + p.eps);
    T* y = reinterpret_cast<T*>(p.y) + ((long long)s * p.T + rr) * p.y_ld + h * p.vdim + e0;
    const float* nw = p.norm + h * p.vdim + e0;
#pragma unroll
    for (int g = 0; g < kMoCols / 32; g++) {
      if (g >= o_groups) break;
      uint32_t o[32];
      tmem_ld_32x32(tmem_o + lane_addr + (uint32_t)(g * 32), o);
      tmem_ld_wait();
      if (row >= p.T) continue;
#pragma unroll
      for (int q = 0; q < 4; q++) {
        const int c0 = g * 32 + q * 8;
        if (c0 >= ne) break;
        const T* zv = reinterpret_cast<const T*>(&z[g * 4 + q]);
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; e++) v[e] = __uint_as_float(o[q * 8 + e]) * rs * __ldg(nw + c0 + e) * __fdividef(1.0f, 1.0f + __expf(-Cvt<T>::to(zv[e])));
        Pack<T> w;
        pack_from_floats<T>(w, v);
        if (a.y_vec) st16(y + c0, w);
        else {
#pragma unroll
          for (int e = 0; e < 8; e++) y[c0 + e] = w.v[e];
        }
      }
    }
    tc_fence_before_sync();
  }
  tc_fence_before_sync();
  __syncwarp();
  if (a.ranks > 1) cluster_sync_all(); else __syncthreads();      // also: no CTA leaves while its sums are being read
  tc_fence_after_sync();
  if (warp == 1) tmem_dealloc(tmem_base_slot, 256);
}

// ── host ────────────────────────────────────────────────────────────────────
static int mt_panels(int n) { return (n + kMtPanel - 1) / kMtPanel; }
// stages of the key and value rings: as much as fits half an SM where two value stages do
static bool mo_stages(int pd, int pv, int* ks, int* vs, int* smem) {
  const int q = pd * 2 * kMtPanelBytes, most = kMtSmemMax - 6 * 1024;
  *ks = 2;
  for (int limit : {107 * 1024, most}) {
    *vs = (limit - 1024 - q - *ks * pd * kMtPanelBytes) / (pv * kMtPanelBytes);
    if (*vs >= 2) break;
  }
  if (*vs > kMoMaxStages) *vs = kMoMaxStages;
  *smem = q + (*ks * pd + *vs * pv) * kMtPanelBytes + 1024;
  return *vs >= 2;
}
static int mo_panels(int vdim) { return vdim >= kMoCols ? 2 : mt_panels(vdim); }

bool mlstm_tc_eligible(const MlstmDesc& d) {
  if (!(d.dtype == DType::BF16 || d.dtype == DType::F16)) return false;
  if (d.dim % 8 || d.vdim % 8 || d.dim > 256 || d.vdim > 8 * kMoCols || d.ld % 8 || !aligned16(d.proj)) return false;
  int ks, vs, smem;
  return mo_stages(mt_panels(d.dim), mo_panels(d.vdim), &ks, &vs, &smem) && matmul_status_word() != nullptr;
}

static Status token_map(CUtensorMap* m, DType dt, const MlParams& p, int64_t col, int width, int box_rows) {
  const uint8_t* base = static_cast<const uint8_t*>(p.proj) + (size_t)col * 2;
  return make_map(m, dt, base, (uint64_t)width, (uint64_t)p.T, (uint64_t)p.heads, (uint64_t)p.n_seq, (uint64_t)p.ld, (uint64_t)width, (uint64_t)p.T * p.ld, kMtPanel, (uint32_t)box_rows);
}

template <typename T>
static cudaError_t launch_mc(cudaStream_t s, const CUtensorMap& mk, const CUtensorMap& mv, const MlChunkTc& a, dim3 grid, size_t smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(ml_chunk_tc_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMtSmemMax - 8 * 1024);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  return launch_pdl(ml_chunk_tc_kernel<T>, grid, dim3(192), smem, s, mk, mv, a);
}
Status mlstm_chunk_tc(cudaStream_t s, DType dt, const MlParams& p) {
  CUtensorMap mk, mv;
  AG_RETURN_IF_ERROR(token_map(&mk, dt, p, (int64_t)p.heads * p.dim, p.dim, kMtTok));
  AG_RETURN_IF_ERROR(token_map(&mv, dt, p, 2 * (int64_t)p.heads * p.dim, p.vdim, kMtTok));
  MlChunkTc a;
  a.p = p; a.m_tiles = (p.dim + 127) / 128; a.n_tiles = (p.vdim + 255) / 256; a.pv = p.vdim > 256 ? 4 : mt_panels(p.vdim); a.status = matmul_status_word();
  const size_t smem = (size_t)kMcStages * (4 + a.pv) * kMtPanelBytes + 1024;
  const dim3 grid((unsigned)(p.w.chunks * a.m_tiles * a.n_tiles), (unsigned)(p.n_seq * p.heads));
  const cudaError_t e = dt == DType::BF16 ? launch_mc<__nv_bfloat16>(s, mk, mv, a, grid, smem) : launch_mc<__half>(s, mk, mv, a, grid, smem);
  return cuda_status(e, "mlstm chunk states (tcgen05)");
}

template <typename T>
static cudaError_t launch_mo(cudaStream_t s, const CUtensorMap* m, const MlOutTc& a, dim3 grid, size_t smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(ml_output_tc_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMtSmemMax - 6 * 1024);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid; cfg.blockDim = dim3(192); cfg.dynamicSmemBytes = smem; cfg.stream = s;
  cudaLaunchAttribute at[2];
  at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization; at[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  at[1].id = cudaLaunchAttributeClusterDimension; at[1].val.clusterDim.x = (unsigned)a.ranks; at[1].val.clusterDim.y = 1; at[1].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = a.ranks > 1 ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, ml_output_tc_kernel<T>, m[0], m[1], m[2], m[3], a);
}
Status mlstm_output_tc(cudaStream_t s, DType dt, const MlParams& p) {
  CUtensorMap m[4];
  AG_RETURN_IF_ERROR(token_map(&m[0], dt, p, 0, p.dim, 128));
  AG_RETURN_IF_ERROR(token_map(&m[1], dt, p, (int64_t)p.heads * p.dim, p.dim, kMtTok));
  AG_RETURN_IF_ERROR(token_map(&m[2], dt, p, 2 * (int64_t)p.heads * p.dim, p.vdim, kMtTok));
  const uint64_t plane = (uint64_t)p.dim * p.vdim;
  AG_RETURN_IF_ERROR(make_map(&m[3], dt, p.w.planes, (uint64_t)p.vdim, (uint64_t)p.dim, (uint64_t)p.w.chunks * 2, (uint64_t)p.n_seq * p.heads, (uint64_t)p.vdim, plane,
                              plane * p.w.chunks * 2, kMtPanel, kMtTok));
  MlOutTc a;
  a.p = p; a.pd = mt_panels(p.dim); a.pv = mo_panels(p.vdim); a.ranks = (p.vdim + kMoCols - 1) / kMoCols; a.status = matmul_status_word();
  a.y_vec = aligned16(p.y) && p.y_ld % 8 == 0 ? 1 : 0;
  int smem = 0;
  if (!mo_stages(a.pd, a.pv, &a.ks, &a.vs, &smem)) return Status::unsupported("mlstm output: head too large");
  const dim3 grid((unsigned)((p.T + 127) / 128 * a.ranks), (unsigned)(p.n_seq * p.heads));
  const cudaError_t e = dt == DType::BF16 ? launch_mo<__nv_bfloat16>(s, m, a, grid, (size_t)smem) : launch_mo<__half>(s, m, a, grid, (size_t)smem);
  return cuda_status(e, "mlstm output (tcgen05)");
}

}}  // namespace ag::k
