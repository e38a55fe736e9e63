// End of a block whose mixer and feed-forward read the same input, fused with the start of the next one (fp32 arithmetic whatever the
// storage types; a type code per tensor; compiled without fast-math):
//
//   R(v)  = v / sqrt(mean(v^2) + eps)
//   res  += (a * (w1 ? R(y1) * w1 : y1) + b * (w2 ? R(y2) * w2 : y2)) + y3 [+ step]      (y1, y2, y3, step optional)
//   out   = R(res) * (w_next + w_off)                                                    (optional)
//
// y1 / y2: the outputs of a mixer's two sides (each with a norm of its own, or none), y3: the feed-forward's, step: a vector added to
// every row (the start of a pass of a loop).  One CTA per row; every reduction runs over a fixed thread-to-element map and a fixed
// tree, so a row's result does not depend on the batch it is in.  Rows of a multiple of 4 elements (up to 8192) with aligned tensors
// stay in registers, four elements per access, all loads issued before the first reduction; both side norms share one reduction
// round.  Other rows go through shared memory, element by element.
#include "anytype.cuh"

namespace {

using rb::ld_any;
using rb::st_any;

constexpr int kThreads = 256;      // of the shared-memory form

struct BranchParams {
  void* res; int dtr;                       // [T, W] updated in place
  const void* y1; const void* y2; const void* y3; int64_t ld1, ld2, ld3; int dty;   // [T, W] each or null
  float a, b;
  const void* w1; const void* w2; const void* step; const void* w_next; int dtw;    // [W] each or null
  float w_off;
  void* out; int dto;                       // [T, W] or null
  int W; float eps;
};

// sums of two values over the CTA (one round); `red` holds >= 32 float2
RB_DEVICE float2 block_sum2(float x, float y, float2* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  x = rb::warp_sum(x);
  y = rb::warp_sum(y);
  __syncthreads();
  if (lane == 0) red[warp] = make_float2(x, y);
  __syncthreads();
  const float2 v = lane < (blockDim.x >> 5) ? red[lane] : make_float2(0.f, 0.f);
  return make_float2(rb::warp_sum(v.x), rb::warp_sum(v.y));
}

RB_DEVICE float inv_rms(float ss, int W, float eps) { return 1.f / sqrtf(ss / (float)W + eps); }
RB_DEVICE float dot4(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }
RB_DEVICE float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }

// NV float4 per thread, NT threads (many threads with few elements each keep more loads in flight than the reverse: four streams are read)
template <int NV, int NT>
__global__ void __launch_bounds__(NT) branch_norm_reg_kernel(BranchParams p) {
  __shared__ float2 red2[32];
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const int W = p.W;
  rb::pdl_trigger();
  rb::pdl_wait();
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 r[NV], m1[NV], m2[NV], f[NV];
  float s1 = 0.f, s2 = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int e = (threadIdx.x + j * NT) * 4;
    r[j] = m1[j] = m2[j] = f[j] = zero;
    if (e < W) {
      r[j] = rb::ld4_any(p.res, p.dtr, t * (int64_t)W + e);
      if (p.y1 != nullptr) m1[j] = rb::ld4_any(p.y1, p.dty, t * p.ld1 + e);
      if (p.y2 != nullptr) m2[j] = rb::ld4_any(p.y2, p.dty, t * p.ld2 + e);
      if (p.y3 != nullptr) f[j] = rb::ld4_any(p.y3, p.dty, t * p.ld3 + e);
    }
  }
#pragma unroll
  for (int j = 0; j < NV; ++j) { s1 += dot4(m1[j]); s2 += dot4(m2[j]); }
  float c1 = p.a, c2 = p.b;
  if (p.w1 != nullptr || p.w2 != nullptr) {
    const float2 s = block_sum2(s1, s2, red2);
    if (p.w1 != nullptr) c1 *= inv_rms(s.x, W, p.eps);
    if (p.w2 != nullptr) c2 *= inv_rms(s.y, W, p.eps);
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int e = (threadIdx.x + j * NT) * 4;
    if (e < W) {
      float4 u = m1[j], v = m2[j];
      if (p.w1 != nullptr) { const float4 w = rb::ld4_any(p.w1, p.dtw, e); u = make_float4(u.x * w.x, u.y * w.y, u.z * w.z, u.w * w.w); }
      if (p.w2 != nullptr) { const float4 w = rb::ld4_any(p.w2, p.dtw, e); v = make_float4(v.x * w.x, v.y * w.y, v.z * w.z, v.w * w.w); }
      const float4 y = make_float4(fmaf(u.x, c1, v.x * c2) + f[j].x, fmaf(u.y, c1, v.y * c2) + f[j].y, fmaf(u.z, c1, v.z * c2) + f[j].z,
                                   fmaf(u.w, c1, v.w * c2) + f[j].w);
      float4 x = add4(r[j], y);
      if (p.step != nullptr) x = add4(x, rb::ld4_any(p.step, p.dtw, e));
      rb::st4_any(p.res, p.dtr, t * (int64_t)W + e, x);
      r[j] = make_float4(rb::round_any(p.dtr, x.x), rb::round_any(p.dtr, x.y), rb::round_any(p.dtr, x.z), rb::round_any(p.dtr, x.w));
      ss += dot4(r[j]);
    }
  }
  if (p.out == nullptr) return;
  const float rs = inv_rms(rb::block_reduce<false>(ss, red), W, p.eps);
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int e = (threadIdx.x + j * NT) * 4;
    if (e < W) {
      const float4 w = rb::ld4_any(p.w_next, p.dtw, e);
      rb::st4_any(p.out, p.dto, t * (int64_t)W + e, make_float4(r[j].x * rs * (w.x + p.w_off), r[j].y * rs * (w.y + p.w_off), r[j].z * rs * (w.z + p.w_off),
                                                                r[j].w * rs * (w.w + p.w_off)));
    }
  }
}

__global__ void __launch_bounds__(kThreads) branch_norm_kernel(BranchParams p) {
  extern __shared__ float row[];
  __shared__ float2 red2[32];
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const int W = p.W;
  rb::pdl_trigger();
  rb::pdl_wait();
  float s1 = 0.f, s2 = 0.f;
  for (int e = threadIdx.x; e < W; e += kThreads) {
    if (p.w1 != nullptr) { const float v = ld_any(p.y1, p.dty, t * p.ld1 + e); s1 = fmaf(v, v, s1); }
    if (p.w2 != nullptr) { const float v = ld_any(p.y2, p.dty, t * p.ld2 + e); s2 = fmaf(v, v, s2); }
  }
  const float2 s = block_sum2(s1, s2, red2);
  const float c1 = p.w1 != nullptr ? p.a * inv_rms(s.x, W, p.eps) : p.a, c2 = p.w2 != nullptr ? p.b * inv_rms(s.y, W, p.eps) : p.b;
  float ss = 0.f;
  for (int e = threadIdx.x; e < W; e += kThreads) {     // every thread re-reads only the elements it wrote
    float u = p.y1 != nullptr ? ld_any(p.y1, p.dty, t * p.ld1 + e) : 0.f, v = p.y2 != nullptr ? ld_any(p.y2, p.dty, t * p.ld2 + e) : 0.f;
    if (p.w1 != nullptr) u *= ld_any(p.w1, p.dtw, e);
    if (p.w2 != nullptr) v *= ld_any(p.w2, p.dtw, e);
    float y = fmaf(u, c1, v * c2);
    if (p.y3 != nullptr) y += ld_any(p.y3, p.dty, t * p.ld3 + e);
    float x = ld_any(p.res, p.dtr, t * (int64_t)W + e) + y;
    if (p.step != nullptr) x += ld_any(p.step, p.dtw, e);
    st_any(p.res, p.dtr, t * (int64_t)W + e, x);
    x = rb::round_any(p.dtr, x);
    row[e] = x;
    ss = fmaf(x, x, ss);
  }
  if (p.out == nullptr) return;
  const float rs = inv_rms(rb::block_reduce<false>(ss, red), W, p.eps);
  for (int e = threadIdx.x; e < W; e += kThreads) st_any(p.out, p.dto, t * (int64_t)W + e, row[e] * rs * (ld_any(p.w_next, p.dtw, e) + p.w_off));
}

inline bool al16(const void* q) { return q == nullptr || (reinterpret_cast<uintptr_t>(q) & 15) == 0; }
inline bool al_ld(const void* q, int64_t ld) { return q == nullptr || ld % 4 == 0; }

}  // namespace

// res [T, W] (type dtr); y1 / y2 / y3 rows of stride ld1 / ld2 / ld3 (type dty); w1 needs y1, w2 needs y2; the vectors share type dtw
extern "C" int rb_branch_norm(void* res, int dtr, const void* y1, int64_t ld1, const void* y2, int64_t ld2, const void* y3, int64_t ld3, int dty,
                              float a, float b, const void* w1, const void* w2, const void* step, const void* w_next, int dtw, float w_off, void* out,
                              int dto, int64_t T, int W, float eps, cudaStream_t s) {
  if (T == 0) return 0;
  if (W < 1 || res == nullptr || (w1 != nullptr && y1 == nullptr) || (w2 != nullptr && y2 == nullptr) || ((out == nullptr) != (w_next == nullptr))) return -1;
  BranchParams p{res, dtr, y1, y2, y3, ld1, ld2, ld3, dty, a, b, w1, w2, step, w_next, dtw, w_off, out, dto, W, eps};
  const bool vec = W % 4 == 0 && W <= 8192 && al_ld(y1, ld1) && al_ld(y2, ld2) && al_ld(y3, ld3) && al16(res) && al16(y1) && al16(y2) && al16(y3) &&
                   al16(w1) && al16(w2) && al16(step) && al16(w_next) && al16(out);
  if (vec) {
    auto kern = W <= 1024 ? branch_norm_reg_kernel<1, 256> : W <= 2048 ? branch_norm_reg_kernel<1, 512> : W <= 4096 ? branch_norm_reg_kernel<1, 1024>
                                                                                                        : branch_norm_reg_kernel<2, 1024>;
    const int nt = W <= 1024 ? 256 : W <= 2048 ? 512 : 1024;
    return rb::launch_pdl(kern, dim3((unsigned)T), dim3(nt), 0, s, p) == cudaSuccess ? 0 : 2;
  }
  const size_t smem = (size_t)W * sizeof(float);
  if (smem > 160 * 1024) return -1;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(branch_norm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return 2;
  return rb::launch_pdl(branch_norm_kernel, dim3((unsigned)T), dim3(kThreads), smem, s, p) == cudaSuccess ? 0 : 2;
}
