// Linears of a step that carries at most 16 rows (a generated token per sequence, or a prompt portion of a few tokens).
//
// Such a product is bound by reading its K-major weight once. 16-bit models take the tensor-core form further down. In the other
// one, a warp owns RW weight rows (for the gated form RW / 2
// gate rows and their up rows), its lanes split K in 16-byte pieces, and the input rows wait in shared memory as floats.
// One launch serves up to three weights that read the same stream: the projections of a mixer and of the feed-forward
// beside it depend on nothing but x, so a layer starts with a single launch whose prologue takes the RMS norms. The
// float32 residual is updated in the epilogue of the output product.
#include "common.cuh"
#include "seq_kernels.h"
#include "mma_sync.cuh"
#include "sm100.cuh"

namespace ag { namespace k {

constexpr int kSsThreads = 256;
constexpr int kSsWarps = kSsThreads / 32;
constexpr size_t kSsMaxSmem = 200 * 1024;

struct SsSeg {
  const void* w; void* out; const float* norm_w;
  long long ld, out_ld;
  int n, mode, glu, block0;          // block0: first block of this segment
  float limit;
};
struct SsParams {
  const float* x; const void* a; long long a_ld; float eps;
  int rows, k, kp, n_seg;            // kp: k rounded up to whole 8-element packs (the weights hold zeros there)
  SsSeg seg[kSeqSegs];
};

template <typename T, int MR, int RW>
__global__ void __launch_bounds__(kSsThreads) seq_skinny_kernel(const SsParams p) {
  extern __shared__ __align__(16) float s_in[];       // [MR][kp]
  constexpr int VEC = 16 / (int)sizeof(T);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int si = 0;
#pragma unroll
  for (int i = 1; i < kSeqSegs; i++) if (i < p.n_seg && (int)blockIdx.x >= p.seg[i].block0) si = i;
  const SsSeg sg = p.seg[si];
  const bool glu = sg.mode == (int)SeqOut::Glu;
  constexpr int GW = RW >= 2 ? RW / 2 : 1;
  const int n0 = (((int)blockIdx.x - sg.block0) * kSsWarps + warp) * (glu ? GW : RW);
  const T* W = reinterpret_cast<const T*>(sg.w);
  // weight row of register slot r: gate rows in the first half of the slots, the rows of the values they gate in the second
  auto row_of = [&](int r) -> long long {
    if (!glu) return n0 + r < sg.n ? n0 + r : -1;
    const int c = n0 + r % GW;
    return c < sg.n ? (long long)(c / kGluBlock * 2 * kGluBlock + c % kGluBlock + r / GW * kGluBlock) : -1;
  };
  const T* wp[RW];
#pragma unroll
  for (int r = 0; r < RW; r++) { const long long q = row_of(r); wp[r] = q < 0 ? nullptr : W + q * sg.ld; }
  // model weights are not written by the step: start them towards the L2 before waiting for the previous kernel
#pragma unroll
  for (int r = 0; r < RW; r++)
    if (wp[r]) for (int kc = lane * 128 / (int)sizeof(T); kc < p.kp; kc += 32 * 128 / (int)sizeof(T)) asm volatile("prefetch.global.L2 [%0];" ::"l"(wp[r] + kc));
  pdl_wait();
  pdl_trigger();
  const int m0 = (int)blockIdx.y * MR;
  const int mrows = min(MR, p.rows - m0);
  if (p.x) {
    for (int m = warp; m < MR; m += kSsWarps) {
      float* dst = s_in + (long long)m * p.kp;
      if (m >= mrows) { for (int c = lane; c < p.kp; c += 32) dst[c] = 0.f; continue; }
      const float* xr = p.x + (long long)(m0 + m) * p.k;
      float sq = 0.f;
      for (int c = lane; c < p.kp; c += 32) { const float v = c < p.k ? xr[c] : 0.f; dst[c] = v; sq = fmaf(v, v, sq); }
      const float rs = 1.0f / sqrtf(warp_sum(sq) / (float)p.k + p.eps);
      for (int c = lane; c < p.k; c += 32) dst[c] *= rs * sg.norm_w[c];
    }
  } else {
    const T* A = reinterpret_cast<const T*>(p.a);
    for (int i = threadIdx.x; i < MR * p.kp; i += kSsThreads) {
      const int m = i / p.kp, c = i - m * p.kp;
      s_in[i] = (m < mrows && c < p.k) ? Cvt<T>::to(A[(long long)(m0 + m) * p.a_ld + c]) : 0.f;
    }
  }
  __syncthreads();
  if (n0 >= sg.n) return;
  float acc[MR][RW];
#pragma unroll
  for (int m = 0; m < MR; m++)
#pragma unroll
    for (int r = 0; r < RW; r++) acc[m][r] = 0.f;
#pragma unroll 2
  for (int kc = lane * VEC; kc < p.kp; kc += 32 * VEC) {
    Pack<T> raw[RW];
#pragma unroll
    for (int r = 0; r < RW; r++) {
      if (wp[r]) raw[r] = ld16_stream(wp[r] + kc);
      else {
#pragma unroll
        for (int e = 0; e < VEC; e++) raw[r].v[e] = Cvt<T>::from(0.f);
      }
    }
#pragma unroll
    for (int m = 0; m < MR; m++) {
      float af[VEC];
#pragma unroll
      for (int q = 0; q < VEC / 4; q++) {
        const float4 a4 = *reinterpret_cast<const float4*>(s_in + (long long)m * p.kp + kc + q * 4);
        af[q * 4] = a4.x; af[q * 4 + 1] = a4.y; af[q * 4 + 2] = a4.z; af[q * 4 + 3] = a4.w;
      }
#pragma unroll
      for (int r = 0; r < RW; r++)
#pragma unroll
        for (int e = 0; e < VEC; e++) acc[m][r] = fmaf(af[e], Cvt<T>::to(raw[r].v[e]), acc[m][r]);
    }
  }
#pragma unroll
  for (int m = 0; m < MR; m++)
#pragma unroll
    for (int r = 0; r < RW; r++) acc[m][r] = warp_sum(acc[m][r]);
  // every lane holds all sums; lane l finishes results l, l + 32, ...
#pragma unroll
  for (int m = 0; m < MR; m++) {
    if (m >= mrows) continue;
    const long long row = m0 + m;
    if (glu) {
      if constexpr (RW >= 2) {
#pragma unroll
        for (int r = 0; r < GW; r++) {
          if (((m * GW + r) & 31) != lane || n0 + r >= sg.n) continue;
          reinterpret_cast<T*>(sg.out)[row * sg.out_ld + n0 + r] = Cvt<T>::from(glu_f(sg.glu, acc[m][r], acc[m][GW + r], sg.limit));
        }
      }
      continue;
    }
#pragma unroll
    for (int r = 0; r < RW; r++) {
      if (((m * RW + r) & 31) != lane || n0 + r >= sg.n) continue;
      const long long o = row * sg.out_ld + n0 + r;
      if (sg.mode == (int)SeqOut::Store) reinterpret_cast<T*>(sg.out)[o] = Cvt<T>::from(acc[m][r]);
      else if (sg.mode == (int)SeqOut::StoreF32) reinterpret_cast<float*>(sg.out)[o] = acc[m][r];
      else reinterpret_cast<float*>(sg.out)[o] += acc[m][r];
    }
  }
}

// ── the tensor-core form ────────────────────────────────────────────────────
// 16-bit weights and inputs. A CTA owns 16 weight rows (for the gated form 8 gate rows and the 8 rows they gate), its eight
// warps take every eighth 32-column block of K, and mma.m16n8k16 multiplies them with the input rows as the 8-wide
// operand. The order of K inside a block is free as long as both operands agree on it, so a lane feeds two MMAs from one
// 16-byte piece of each of its two weight rows and of its input row: no shared memory and no shuffles in the loop. The
// first pieces of the weights are requested before the programmatic dependency wait. The warps' sums meet in shared memory;
// a product with few result columns and long rows spreads K over a cluster, whose sums meet over distributed shared memory.
struct SmSeg { const void* w; const void* a; void* out; long long ld, a_ld, out_ld; int n, mode, glu, block0; float limit; };
struct SmParams { SmSeg seg[kSeqSegs]; int n_seg, rows, kp, ranks; };       // ranks: CTAs of a cluster along K

template <typename T, int NT>        // NT groups of 8 input rows
__global__ void __launch_bounds__(kSsThreads) seq_skinny_mma_kernel(const SmParams p) {
  constexpr int U = 4;               // 32-column blocks in flight per warp
  __shared__ float red[kSsWarps][NT * 8][17];
  __shared__ float part[NT * 8][16];
  const int rank = p.ranks > 1 ? (int)sm100::cluster_ctarank() : 0, stride = kSsWarps * p.ranks;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  int si = 0;
#pragma unroll
  for (int i = 1; i < kSeqSegs; i++) if (i < p.n_seg && (int)(blockIdx.x / p.ranks) >= p.seg[i].block0) si = i;
  const SmSeg sg = p.seg[si];
  const bool glu = sg.mode == (int)SeqOut::Glu;
  const int group = (int)(blockIdx.x / p.ranks) - sg.block0;
  const int c0 = group * (glu ? 8 : 16);                        // first result column
  long long r0, r1;                                             // this lane's two weight rows
  if (glu) { r0 = c0 / kGluBlock * 2 * kGluBlock + c0 % kGluBlock + g; r1 = r0 + kGluBlock; }
  else { r0 = c0 + g; r1 = r0 + 8; }
  const bool live0 = glu || r0 < sg.n, live1 = glu || r1 < sg.n;
  const T* w0 = reinterpret_cast<const T*>(sg.w) + r0 * sg.ld;
  const T* w1 = reinterpret_cast<const T*>(sg.w) + r1 * sg.ld;
  const T* x[NT];
#pragma unroll
  for (int t = 0; t < NT; t++) x[t] = g + 8 * t < p.rows ? reinterpret_cast<const T*>(sg.a) + (long long)(g + 8 * t) * sg.a_ld : nullptr;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  float acc[NT][4];
#pragma unroll
  for (int t = 0; t < NT; t++) { acc[t][0] = 0.f; acc[t][1] = 0.f; acc[t][2] = 0.f; acc[t][3] = 0.f; }
  uint4 a0[U], a1[U];
  auto fetch = [&](int kb) {
#pragma unroll
    for (int u = 0; u < U; u++) {
      const int kk = (kb + u * stride) * 32 + q * 8;
      a0[u] = live0 && kk < p.kp ? __ldcs(reinterpret_cast<const uint4*>(w0 + kk)) : zero;
      a1[u] = live1 && kk < p.kp ? __ldcs(reinterpret_cast<const uint4*>(w1 + kk)) : zero;
    }
  };
  fetch(rank * kSsWarps + warp);
  pdl_wait();
  pdl_trigger();
  for (int kb = rank * kSsWarps + warp; kb * 32 < p.kp;) {
    uint4 b[U][NT];
#pragma unroll
    for (int u = 0; u < U; u++) {
      const int kk = (kb + u * stride) * 32 + q * 8;
#pragma unroll
      for (int t = 0; t < NT; t++) b[u][t] = x[t] && kk < p.kp ? *reinterpret_cast<const uint4*>(x[t] + kk) : zero;
    }
#pragma unroll
    for (int u = 0; u < U; u++)
#pragma unroll
      for (int t = 0; t < NT; t++) {
        mma_16816<T>(acc[t], a0[u].x, a1[u].x, a0[u].y, a1[u].y, b[u][t].x, b[u][t].y);
        mma_16816<T>(acc[t], a0[u].z, a1[u].z, a0[u].w, a1[u].w, b[u][t].z, b[u][t].w);
      }
    kb += U * stride;
    if (kb * 32 < p.kp) fetch(kb);
  }
#pragma unroll
  for (int t = 0; t < NT; t++) {      // lane: rows g and g + 8 of the weights, input rows 2 q and 2 q + 1
    red[warp][t * 8 + 2 * q][g] = acc[t][0]; red[warp][t * 8 + 2 * q + 1][g] = acc[t][1];
    red[warp][t * 8 + 2 * q][g + 8] = acc[t][2]; red[warp][t * 8 + 2 * q + 1][g + 8] = acc[t][3];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < NT * 8 * 16; i += kSsThreads) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < kSsWarps; w++) v += red[w][i / 16][i % 16];
    part[i / 16][i % 16] = v;
  }
  if (p.ranks > 1) sm100::cluster_sync_all(); else __syncthreads();
  if (rank == 0) {
    auto total = [&](int m, int n) {
      float v = part[m][n];
      for (int r = 1; r < p.ranks; r++) {
        float u;
        asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(u) : "r"(sm100::mapa_u32(sm100::smem_u32(&part[m][n]), (uint32_t)r)));
        v += u;
      }
      return v;
    };
    const int width = glu ? 8 : 16;
    for (int i = threadIdx.x; i < NT * 8 * width; i += kSsThreads) {
      const int m = i / width, n = i % width;
      if (m >= p.rows || c0 + n >= sg.n) continue;
      const float v = total(m, n);
      const long long o = (long long)m * sg.out_ld + c0 + n;
      if (glu) reinterpret_cast<T*>(sg.out)[o] = Cvt<T>::from(glu_f(sg.glu, v, total(m, n + 8), sg.limit));
      else if (sg.mode == (int)SeqOut::Store) reinterpret_cast<T*>(sg.out)[o] = Cvt<T>::from(v);
      else if (sg.mode == (int)SeqOut::StoreF32) reinterpret_cast<float*>(sg.out)[o] = v;
      else reinterpret_cast<float*>(sg.out)[o] += v;
    }
  }
  if (p.ranks > 1) sm100::cluster_sync_all();      // no CTA leaves while its sums are being read
}

template <typename T, int NT>
static cudaError_t launch_sm(cudaStream_t s, const SmParams& p, int blocks) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)(blocks * p.ranks)); cfg.blockDim = dim3(kSsThreads); cfg.stream = s;
  cudaLaunchAttribute at[2];
  at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization; at[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  at[1].id = cudaLaunchAttributeClusterDimension; at[1].val.clusterDim.x = (unsigned)p.ranks; at[1].val.clusterDim.y = 1; at[1].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = p.ranks > 1 ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, seq_skinny_mma_kernel<T, NT>, p);
}

static Status seq_skinny_mma(cudaStream_t s, const SeqSkinnyDesc& d) {
  SmParams p;
  p.n_seg = d.n_seg; p.rows = d.rows; p.kp = (int)pad8(d.k);
  int blocks = 0;
  for (int i = 0; i < d.n_seg; i++) {
    const SeqSeg& g = d.seg[i];
    if (!g.w || !g.out || !g.a || g.n < 1 || g.ld % 8 != 0 || g.ld < d.k || g.a_ld % 8 != 0 || g.a_ld < p.kp || !aligned16(g.w) || !aligned16(g.a)) return Status::invalid("seq_skinny: bad segment");
    SmSeg& q = p.seg[i];
    q.w = g.w; q.a = g.a; q.out = g.out; q.ld = g.ld; q.a_ld = g.a_ld; q.out_ld = g.out_ld; q.n = g.n; q.mode = (int)g.mode; q.glu = (int)g.glu; q.block0 = blocks; q.limit = g.limit;
    const int per = g.mode == SeqOut::Glu ? 8 : 16;
    blocks += (g.n + per - 1) / per;
  }
  p.ranks = 1;                                     // few blocks: more CTAs along K, as long as each warp keeps a full round of it
  while (p.ranks < 4 && blocks * p.ranks < 2 * sm_count() && p.kp / 32 >= kSsWarps * p.ranks * 4) p.ranks *= 2;
  cudaError_t e;
  if (d.dtype == DType::BF16) e = d.rows <= 8 ? launch_sm<__nv_bfloat16, 1>(s, p, blocks) : launch_sm<__nv_bfloat16, 2>(s, p, blocks);
  else e = d.rows <= 8 ? launch_sm<__half, 1>(s, p, blocks) : launch_sm<__half, 2>(s, p, blocks);
  return cuda_status(e, "seq_skinny (tensor cores)");
}

bool seq_skinny_fits(int64_t k) { return pad8(k) * (int64_t)sizeof(float) <= (int64_t)kSsMaxSmem; }

template <typename T, int MR, int RW>
static cudaError_t launch_ss(cudaStream_t s, const SsParams& p, dim3 grid, size_t smem) {
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(seq_skinny_kernel<T, MR, RW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSsMaxSmem);
    if (e != cudaSuccess) return e;
    attr = true;
  }
  return launch_pdl(seq_skinny_kernel<T, MR, RW>, grid, dim3(kSsThreads), smem, s, p);
}
template <typename T, int MR>
static cudaError_t launch_ss_rw(cudaStream_t s, const SsParams& p, dim3 grid, size_t smem, int rw) {
  return rw == 4 ? launch_ss<T, MR, 4>(s, p, grid, smem) : launch_ss<T, MR, 2>(s, p, grid, smem);
}

Status seq_skinny(cudaStream_t s, const SeqSkinnyDesc& d) {
  if (d.rows < 1 || d.rows > kSeqSkinnyRows || d.n_seg < 1 || d.n_seg > kSeqSegs) return Status::invalid("seq_skinny: bad description");
  if (d.seg[0].a && d.dtype != DType::F32) return seq_skinny_mma(s, d);
  if (!d.x == !d.a) return Status::invalid("seq_skinny: one input");
  if (!seq_skinny_fits(d.k)) return Status::unsupported("seq_skinny: input rows too long");
  SsParams p;
  p.x = d.x; p.a = d.a; p.a_ld = d.a_ld; p.eps = d.eps; p.rows = d.rows; p.k = d.k; p.kp = (int)pad8(d.k); p.n_seg = d.n_seg;
  int mr = 1;
  while (mr < d.rows && (size_t)(2 * mr) * p.kp * sizeof(float) <= kSsMaxSmem) mr *= 2;
  int64_t total = 0;
  for (int i = 0; i < d.n_seg; i++) total += d.seg[i].n * (d.seg[i].mode == SeqOut::Glu ? 2 : 1);
  const int rw = total / 4 >= (int64_t)sm_count() * 16 ? 4 : 2;    // enough warps to fill the machine either way
  int blocks = 0;
  for (int i = 0; i < d.n_seg; i++) {
    const SeqSeg& g = d.seg[i];
    if (!g.w || !g.out || g.n < 1 || g.ld % 8 != 0 || g.ld < d.k || !aligned16(g.w) || (d.x && !g.norm_w)) return Status::invalid("seq_skinny: bad segment");
    SsSeg& q = p.seg[i];
    q.w = g.w; q.out = g.out; q.norm_w = g.norm_w; q.ld = g.ld; q.out_ld = g.out_ld; q.n = g.n; q.mode = (int)g.mode; q.glu = (int)g.glu; q.limit = g.limit; q.block0 = blocks;
    const int per = (g.mode == SeqOut::Glu ? rw / 2 : rw) * kSsWarps;
    blocks += (g.n + per - 1) / per;
  }
  const size_t smem = (size_t)mr * p.kp * sizeof(float);
  dim3 grid((unsigned)blocks, (unsigned)((d.rows + mr - 1) / mr));
  cudaError_t e = cudaSuccess;
  AG_DISPATCH_FLOAT(d.dtype, T, {
    switch (mr) {
      case 1: e = launch_ss_rw<T, 1>(s, p, grid, smem, rw); break;
      case 2: e = launch_ss_rw<T, 2>(s, p, grid, smem, rw); break;
      case 4: e = launch_ss_rw<T, 4>(s, p, grid, smem, rw); break;
      case 8: e = launch_ss_rw<T, 8>(s, p, grid, smem, rw); break;
      default: e = launch_ss_rw<T, 16>(s, p, grid, smem, rw); break;
    }
  });
  return cuda_status(e, "seq_skinny");
}

__global__ void seq_advance_kernel(int* pos, int n_seq, int T, const int32_t* tok, int32_t* history, int* step, int max_steps) {
  pdl_wait();
  pdl_trigger();
  const int st = history ? *step : 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n_seq; i += blockDim.x) {
    pos[i] += T;
    if (history && st < max_steps) history[(long long)st * n_seq + i] = tok[i];
  }
  if (history && threadIdx.x == 0) *step = st + 1;
}
Status seq_advance(cudaStream_t s, int* pos, int n_seq, int T, const int32_t* tok, int32_t* history, int* step, int max_steps) {
  cudaError_t e = launch_pdl(seq_advance_kernel, dim3(1), dim3(128), 0, s, pos, n_seq, T, tok, history, step, max_steps);
  return cuda_status(e, "seq_advance");
}

}}  // namespace ag::k
