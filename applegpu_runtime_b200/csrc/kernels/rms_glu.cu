// RMS norms over a float32 residual stream and the gated activations of a feed-forward.
//
// rms_rows is the only kernel that touches the stream between two layers: it starts it from the embedding table, adds
// what a repeated pass adds ahead of its first layer (the embedding output and a step vector), and writes the two
// normalised copies a parallel layer feeds to its mixer and its feed-forward, all in one pass over the row.
#include "common.cuh"
#include "seq_kernels.h"

namespace ag { namespace k {

constexpr int kRmsThreads = 128;      // small blocks: many rows in flight per SM

struct RmsParams {
  float* x; const int32_t* tok; const void* embed; const float* step; const float* post; const float* wp; const float* w1; const float* w2; const int32_t* row_map;
  void* out1; void* out2;
  long long ld1, ld2, embed_ld;
  int width, vocab, load_x, write_x;
  float eps, embed_scale;
};

// VEC elements per thread and access (4 when width and pitches allow it), NREG accesses kept in registers (wider rows are read
// twice)
template <typename T, int VEC, int NREG>
__global__ void __launch_bounds__(kRmsThreads) rms_rows_kernel(const RmsParams p) {
  __shared__ float red[33];
  pdl_wait();
  pdl_trigger();
  const long long r = blockIdx.x;
  const long long src = p.row_map ? p.row_map[r] : r;
  float* x = p.x + src * p.width;
  const T* e = nullptr;
  if (p.embed) {
    int t = p.tok[r];
    t = t < 0 ? 0 : (t >= p.vocab ? p.vocab - 1 : t);
    e = reinterpret_cast<const T*>(p.embed) + (long long)t * p.embed_ld;
  }
  float v[NREG][VEC];
  float sq = 0.f;
  const int packs = p.width / VEC;
  const float* y = p.post ? p.post + src * p.width : nullptr;
  float rs_y = 0.f;
  if (y) {                                               // the sublayer's output meets the stream through a norm of its own
    float sy = 0.f;
    for (int i = threadIdx.x; i < packs; i += kRmsThreads) {
      const int c = i * VEC;
      if constexpr (VEC == 4) {
        const float4 q = *reinterpret_cast<const float4*>(y + c);
        sy = fmaf(q.x, q.x, fmaf(q.y, q.y, fmaf(q.z, q.z, fmaf(q.w, q.w, sy))));
      } else sy = fmaf(y[c], y[c], sy);
    }
    rs_y = 1.0f / sqrtf(block_sum(sy, red) / (float)p.width + p.eps);
  }
  auto fetch = [&](int i, float (&o)[VEC]) {
    const int c = i * VEC;
    if (p.load_x) {
      if constexpr (VEC == 4) { const float4 q = *reinterpret_cast<const float4*>(x + c); o[0] = q.x; o[1] = q.y; o[2] = q.z; o[3] = q.w; }
      else o[0] = x[c];
    } else {
#pragma unroll
      for (int j = 0; j < VEC; j++) o[j] = 0.f;
    }
    if (e) {
      alignas(16) T t[VEC];
      if constexpr (VEC == 4 && sizeof(T) == 2) *reinterpret_cast<uint2*>(t) = *reinterpret_cast<const uint2*>(e + c);
      else if constexpr (VEC == 4) *reinterpret_cast<uint4*>(t) = *reinterpret_cast<const uint4*>(e + c);
      else t[0] = e[c];
#pragma unroll
      for (int j = 0; j < VEC; j++) o[j] += Cvt<T>::to(t[j]) * p.embed_scale;
    }
    if (y) {
      float yv[VEC];
      if constexpr (VEC == 4) { const float4 q = *reinterpret_cast<const float4*>(y + c); yv[0] = q.x; yv[1] = q.y; yv[2] = q.z; yv[3] = q.w; }
      else yv[0] = y[c];
#pragma unroll
      for (int j = 0; j < VEC; j++) o[j] += yv[j] * rs_y * __ldg(p.wp + c + j);
    }
    if (p.step) {
#pragma unroll
      for (int j = 0; j < VEC; j++) o[j] += p.step[c + j];
    }
  };
  auto put = [&](int i, const float (&o)[VEC]) {
    const int c = i * VEC;
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(x + c) = make_float4(o[0], o[1], o[2], o[3]);
    else x[c] = o[0];
  };
#pragma unroll
  for (int it = 0; it < NREG; it++) {
    const int i = threadIdx.x + it * kRmsThreads;
    if (i < packs) {
      fetch(i, v[it]);
      if (p.write_x) put(i, v[it]);
#pragma unroll
      for (int j = 0; j < VEC; j++) sq = fmaf(v[it][j], v[it][j], sq);
    }
  }
  for (int i = threadIdx.x + NREG * kRmsThreads; i < packs; i += kRmsThreads) {   // rows too wide for the registers
    float o[VEC];
    fetch(i, o);
    if (p.write_x) put(i, o);
#pragma unroll
    for (int j = 0; j < VEC; j++) sq = fmaf(o[j], o[j], sq);
  }
  if (!p.out1) return;
  const float rs = 1.0f / sqrtf(block_sum(sq, red) / (float)p.width + p.eps);
  T* o1 = reinterpret_cast<T*>(p.out1) + r * p.ld1;
  T* o2 = p.out2 ? reinterpret_cast<T*>(p.out2) + r * p.ld2 : nullptr;
  auto emit = [&](int i, const float (&o)[VEC]) {
    const int c = i * VEC;
    auto one = [&](T* dst, const float* w) {
      alignas(16) T t[VEC];
#pragma unroll
      for (int j = 0; j < VEC; j++) t[j] = Cvt<T>::from(o[j] * rs * __ldg(w + c + j));
      if constexpr (VEC == 4 && sizeof(T) == 4) *reinterpret_cast<uint4*>(dst + c) = *reinterpret_cast<const uint4*>(t);
      else if constexpr (VEC == 4) *reinterpret_cast<uint2*>(dst + c) = *reinterpret_cast<const uint2*>(t);
      else dst[c] = t[0];
    };
    one(o1, p.w1);
    if (o2) one(o2, p.w2);
  };
#pragma unroll
  for (int it = 0; it < NREG; it++) {
    const int i = threadIdx.x + it * kRmsThreads;
    if (i < packs) emit(i, v[it]);
  }
  for (int i = threadIdx.x + NREG * kRmsThreads; i < packs; i += kRmsThreads) {
    float o[VEC];
    if (p.write_x) {                                                 // the sum is in x already
#pragma unroll
      for (int j = 0; j < VEC; j++) o[j] = x[i * VEC + j];
    } else fetch(i, o);
    emit(i, o);
  }
}

Status rms_rows(cudaStream_t s, const RmsRowsDesc& d) {
  if (d.rows <= 0) return Status::OK();
  if (d.width < 1 || !d.x || (d.embed && !d.tok) || (d.out1 && !d.w1) || (d.out2 && !d.w2) || (d.post && !d.post_w)) return Status::invalid("rms_rows: missing operand");
  if (d.row_map && (d.embed || d.step || !d.load_x)) return Status::invalid("rms_rows: a gathered row is read only");
  RmsParams p;
  p.x = d.x; p.tok = d.tok; p.embed = d.embed; p.step = d.step; p.post = d.post; p.wp = d.post_w; p.embed_scale = d.embed_scale; p.w1 = d.w1; p.w2 = d.w2; p.row_map = d.row_map;
  p.out1 = d.out1; p.out2 = d.out2; p.ld1 = d.ld1; p.ld2 = d.ld2; p.embed_ld = d.embed_ld;
  p.width = d.width; p.vocab = d.vocab; p.load_x = d.load_x ? 1 : 0; p.write_x = (!d.load_x || d.embed || d.step || (d.post && !d.row_map)) ? 1 : 0; p.eps = d.eps;
  const bool vec = d.width % 4 == 0 && d.ld1 % 4 == 0 && d.ld2 % 4 == 0 && aligned16(d.x) && (!d.post || aligned16(d.post)) && (!d.embed || (d.embed_ld % 4 == 0 && aligned16(d.embed))) && (!d.out1 || aligned16(d.out1)) && (!d.out2 || aligned16(d.out2));
  cudaError_t e = cudaSuccess;
  AG_DISPATCH_FLOAT(d.dtype, T, {
    const dim3 grid((unsigned)d.rows), block(kRmsThreads);
    if (!vec) e = launch_pdl(rms_rows_kernel<T, 1, 16>, grid, block, 0, s, p);
    else if (d.width <= 2 * 4 * kRmsThreads) e = launch_pdl(rms_rows_kernel<T, 4, 2>, grid, block, 0, s, p);
    else if (d.width <= 4 * 4 * kRmsThreads) e = launch_pdl(rms_rows_kernel<T, 4, 4>, grid, block, 0, s, p);
    else if (d.width <= 8 * 4 * kRmsThreads) e = launch_pdl(rms_rows_kernel<T, 4, 8>, grid, block, 0, s, p);
    else e = launch_pdl(rms_rows_kernel<T, 4, 16>, grid, block, 0, s, p);
  });
  return cuda_status(e, "rms_rows");
}

// ── gated activation ────────────────────────────────────────────────
// gate of column c at (c / block) * 2 * block + c % block, the value it gates `block` columns later
template <typename T, int VEC>
__global__ void __launch_bounds__(256) glu_kernel(const T* __restrict__ gu, long long ld_in, T* __restrict__ out, long long ld_out, long long rows, int ff, int block, int kind, float limit) {
  pdl_wait();
  pdl_trigger();
  const int packs = ff / VEC;
  const long long total = rows * packs;
  for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < total; i += (long long)gridDim.x * 256) {
    const long long r = i / packs;
    const int c = (int)(i - r * packs) * VEC;
    const T* g = gu + r * ld_in + c / block * 2 * block + c % block;
    if constexpr (VEC > 1) {
      const Pack<T> a = ld16(g), b = ld16(g + block);
      Pack<T> o;
      float t[VEC];
#pragma unroll
      for (int j = 0; j < VEC; j++) t[j] = glu_f(kind, Cvt<T>::to(a.v[j]), Cvt<T>::to(b.v[j]), limit);
      pack_from_floats<T>(o, t);
      st16(out + r * ld_out + c, o);
    } else {
      out[r * ld_out + c] = Cvt<T>::from(glu_f(kind, Cvt<T>::to(g[0]), Cvt<T>::to(g[block]), limit));
    }
  }
}

Status glu(cudaStream_t s, DType dt, const void* gu, int64_t ld_in, void* out, int64_t ld_out, int64_t rows, int ff, int block, Glu kind, float limit) {
  if (rows <= 0 || ff <= 0) return Status::OK();
  if (block < 1) return Status::invalid("glu: block");
  cudaError_t e = cudaSuccess;
  AG_DISPATCH_FLOAT(dt, T, {
    constexpr int N = Pack<T>::N;
    const bool vec = ff % N == 0 && block % N == 0 && ld_in % N == 0 && ld_out % N == 0 && aligned16(gu) && aligned16(out);
    const int64_t work = rows * (ff / (vec ? N : 1));
    if (vec) e = launch_pdl(glu_kernel<T, N>, dim3((unsigned)grid_for(work, 256)), dim3(256), 0, s, (const T*)gu, (long long)ld_in, (T*)out, (long long)ld_out, (long long)rows, ff, block, (int)kind, limit);
    else e = launch_pdl(glu_kernel<T, 1>, dim3((unsigned)grid_for(work, 256)), dim3(256), 0, s, (const T*)gu, (long long)ld_in, (T*)out, (long long)ld_out, (long long)rows, ff, block, (int)kind, limit);
  });
  return cuda_status(e, "glu");
}

}}  // namespace ag::k
