// What happens to a token's projection row before, and to its attention output after, the attention itself (`WindowAttentionConfig`
// with rotary / full_norm / value_rotary).  fp32 arithmetic with exact sincosf whatever the storage type (compiled without
// fast-math); one CTA per token, whose cos / sin tables (fp32 position x fp32 frequency) are formed once in shared memory.
//
//   window_prepare   row [q (H d) | k (G d) | v (G dv) | ..] in place: q and k divided by their root mean square over ALL their heads
//                    and multiplied by a weight each (wq, wk; null: no norm), the first `dims` dimensions of every q / k head and
//                    the first `vdims` of every v head turned by the position (vdims 0: values untouched).  Packed form: position
//                    pos[t]; cos and sin of q and k carry a factor (`mscale`); with caches the k and v of the tokens a later decode step can still see (the first `keep` positions and
//                    the last rows - keep of the sequence) also go to their cache row (a row without a v section, whose values are its
//                    keys, has one cache).  Step form: position lens[slot of row t]; the
//                    decode kernel stores the row.
//   cache_store      the same call without norm and rotation: the cache rows only
//   turn_gate        attention output [T, H dv] in place: every head turned BACK by the position over its first `dims` columns (the
//                    inverse of the values' rotation), then times sigmoid of a gate logit per head or per element.
//
// Pair layouts: (2i, 2i + 1) or (i, i + dims / 2).  A thread owns whole pairs, four consecutive elements of each half per access when
// sizes and alignment allow (V = 4), else element by element (V = 1).
#include "anytype.cuh"

namespace {

using rb::ld_any;
using rb::st_any;

constexpr int kThreads = 128, kMaxHalf = 512;

template <int V> RB_DEVICE void ldn(const void* p, int dt, int64_t i, float* f) {
  if constexpr (V == 4) {
    const float4 v = rb::ld4_any(p, dt, i);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  } else {
    f[0] = ld_any(p, dt, i);
  }
}
template <int V> RB_DEVICE void stn(void* p, int dt, int64_t i, const float* f) {
  if constexpr (V == 4) rb::st4_any(p, dt, i, make_float4(f[0], f[1], f[2], f[3]));
  else st_any(p, dt, i, f[0]);
}

RB_DEVICE float sig(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }   // fp32 accuracy (a few ulp)

RB_DEVICE int row_position(const int* pos, const int* lens, const int* slots, int64_t t) {
  if (pos != nullptr) return pos[t];
  return lens[slots != nullptr ? slots[t] : t];
}

RB_DEVICE void fill_table(float* cs, float* sn, float p, const float* freq, int half, float mscale = 1.f) {
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(p * freq[i], &s, &c);
    sn[i] = s * mscale;
    cs[i] = c * mscale;
  }
}

// Walks the n_h heads of size hd: f(element offset inside the section, values, n values) after `pre` scaled the loaded elements and the
// pairs turned by +-angle.  `back` turns the other way.
template <int V, typename Pre, typename Out>
RB_DEVICE void walk(const void* x, int dt, int64_t base, int n_h, int hd, int dims, int inter, bool back, const float* cs, const float* sn, Pre pre, Out out) {
  const int half = dims / 2;
  constexpr int P = V == 4 ? 4 : 2;                       // elements of an interleaved unit
  const int rot_units = inter ? dims / P : half / V;
  const int units = rot_units + (hd - dims) / V;
  for (int u = threadIdx.x; u < n_h * units; u += kThreads) {
    const int h = u / units, j = u - h * units;
    if (j >= rot_units) {                                 // untouched by the rotation
      const int e = h * hd + dims + (j - rot_units) * V;
      float a[V];
      ldn<V>(x, dt, base + e, a);
      pre(e, a, V);
      out(e, a, V);
    } else if (inter) {
      const int e0 = j * P, e = h * hd + e0;
      float a[P];
      if constexpr (V == 4) ldn<4>(x, dt, base + e, a);
      else { a[0] = ld_any(x, dt, base + e); a[1] = ld_any(x, dt, base + e + 1); }
      pre(e, a, P);
#pragma unroll
      for (int i = 0; i < P; i += 2) {
        const float c = cs[(e0 + i) >> 1], s = back ? -sn[(e0 + i) >> 1] : sn[(e0 + i) >> 1];
        const float p = a[i], q = a[i + 1];
        a[i] = p * c - q * s;
        a[i + 1] = q * c + p * s;
      }
      out(e, a, P);
    } else {
      const int e0 = j * V, e = h * hd + e0;
      float a[V], b[V];
      ldn<V>(x, dt, base + e, a);
      ldn<V>(x, dt, base + e + half, b);
      pre(e, a, V);
      pre(e + half, b, V);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        const float c = cs[e0 + i], s = back ? -sn[e0 + i] : sn[e0 + i];
        const float p = a[i], q = b[i];
        a[i] = p * c - q * s;
        b[i] = q * c + p * s;
      }
      out(e, a, V);
      out(e + half, b, V);
    }
  }
}

struct PrepareParams {
  void* x; int64_t ld; int dt;
  const void* wq; const void* wk;
  const float* freq; const float* vfreq;
  const int* pos; const int* lens; const int* slots;
  const int* tok_slot; const int* remain;
  void* kc; void* vc;
  int H, G, d, dv, dims, inter, vdims, vinter, keep, rows;
  float eps, mscale;
};

template <int V>
__global__ void __launch_bounds__(kThreads) window_prepare_kernel(PrepareParams p) {
  __shared__ float cs[kMaxHalf], sn[kMaxHalf], vcs[kMaxHalf], vsn[kMaxHalf];
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const int dt = p.dt, nq = p.H * p.d, nk = p.G * p.d;
  rb::pdl_trigger();
  rb::pdl_wait();
  const int n = row_position(p.pos, p.lens, p.slots, t);
  fill_table(cs, sn, (float)n, p.freq, p.dims / 2, p.mscale);
  fill_table(vcs, vsn, (float)n, p.vfreq, p.vdims / 2);
  int64_t slot = -1;
  int row = 0;
  if (p.kc != nullptr) {
    slot = p.tok_slot[t];
    const int ring = max(p.rows - p.keep, 1);
    if (slot >= 0 && !(n < p.keep || p.remain[t] < p.rows - p.keep)) slot = -1;   // a row that a later position of this prompt overwrites
    row = n < p.keep ? n : p.keep + (n - p.keep) % ring;
  }
  const int64_t base = t * p.ld;
  float rq = 1.f, rk = 1.f;
  if (p.wq != nullptr) {
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x * V; c < nq + nk; c += kThreads * V) {
      float a[V];
      ldn<V>(p.x, dt, base + c, a);
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < V; ++i) s += a[i] * a[i];
      if (c < nq) sq += s; else sk += s;
    }
    sq = rb::block_reduce<false>(sq, red);
    sk = rb::block_reduce<false>(sk, red);
    rq = 1.f / sqrtf(sq / (float)nq + p.eps);
    rk = 1.f / sqrtf(sk / (float)nk + p.eps);
  }
  __syncthreads();
  auto norm = [&](const void* w, float r) {
    return [=](int e, float* a, int m) {
      if (w == nullptr) return;
      for (int i = 0; i < m; ++i) a[i] *= r * ld_any(w, dt, e + i);
    };
  };
  // element e of a section -> the row itself and, for keys and values, the token's cache row
  auto emit = [&](int64_t b0, void* cache, int hd) {
    return [=](int e, const float* a, int m) {
      const int64_t i0 = b0 + e;
      const int64_t c0 = cache == nullptr ? 0 : ((slot * p.G + e / hd) * p.rows + row) * hd + e % hd;
      if (m == 4) {
        stn<4>(p.x, dt, i0, a);
        if (cache != nullptr) stn<4>(cache, dt, c0, a);
        return;
      }
      for (int i = 0; i < m; ++i) {
        st_any(p.x, dt, i0 + i, a[i]);
        if (cache != nullptr) st_any(cache, dt, c0 + i, a[i]);
      }
    };
  };
  void* kc = slot >= 0 ? p.kc : nullptr;
  void* vc = slot >= 0 ? p.vc : nullptr;
  if (p.wq != nullptr || p.dims > 0)
    walk<V>(p.x, dt, base, p.H, p.d, p.dims, p.inter, false, cs, sn, norm(p.wq, rq), emit(base, nullptr, p.d));
  if (p.wk != nullptr || p.dims > 0 || kc != nullptr)
    walk<V>(p.x, dt, base + nq, p.G, p.d, p.dims, p.inter, false, cs, sn, norm(p.wk, rk), emit(base + nq, kc, p.d));
  if (p.vdims > 0 || vc != nullptr)
    walk<V>(p.x, dt, base + nq + nk, p.G, p.dv, p.vdims, p.vinter, false, vcs, vsn, norm(nullptr, 1.f), emit(base + nq + nk, vc, p.dv));
}

// Nothing to turn or norm: only the cache rows are written.  A warp per token; tokens that leave no row end at once.
template <int V>
__global__ void __launch_bounds__(kThreads) cache_store_kernel(PrepareParams p, int64_t T) {
  const int64_t t = (int64_t)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
  rb::pdl_trigger();
  rb::pdl_wait();
  if (t >= T) return;
  const int64_t slot = p.tok_slot[t];
  const int n = p.pos[t], ring = max(p.rows - p.keep, 1);
  if (slot < 0 || !(n < p.keep || p.remain[t] < p.rows - p.keep)) return;
  const int row = n < p.keep ? n : p.keep + (n - p.keep) % ring;
  auto copy = [&](int64_t b0, void* cache, int hd) {
    for (int e = (threadIdx.x & 31) * V; e < p.G * hd; e += 32 * V) {
      float a[V];
      ldn<V>(p.x, p.dt, b0 + e, a);
      stn<V>(cache, p.dt, ((slot * p.G + e / hd) * p.rows + row) * hd + e % hd, a);
    }
  };
  const int64_t k0 = t * p.ld + (int64_t)p.H * p.d;
  copy(k0, p.kc, p.d);
  if (p.vc != nullptr) copy(k0 + (int64_t)p.G * p.d, p.vc, p.dv);
}

template <int V>
__global__ void __launch_bounds__(kThreads) turn_gate_kernel(void* __restrict__ x, int dt, const void* __restrict__ gate, int64_t gld, int gmode,
                                                             const float* __restrict__ freq, const int* __restrict__ pos, const int* __restrict__ lens,
                                                             const int* __restrict__ slots, int H, int dv, int dims, int inter) {
  __shared__ float cs[kMaxHalf], sn[kMaxHalf];
  const int64_t t = blockIdx.x;
  rb::pdl_trigger();
  rb::pdl_wait();
  if (dims > 0) {
    fill_table(cs, sn, (float)row_position(pos, lens, slots, t), freq, dims / 2);
    __syncthreads();
  }
  const int64_t base = t * (int64_t)(H * dv);
  walk<V>(x, dt, base, H, dv, dims, inter, true, cs, sn, [](int, float*, int) {},
          [=](int e, float* a, int m) {
            if (gmode == 2 && m == 4) {
              const float4 g = rb::ld4_any(gate, dt, t * gld + e);
              a[0] *= sig(g.x); a[1] *= sig(g.y); a[2] *= sig(g.z); a[3] *= sig(g.w);
            } else if (gmode != 0) {
              for (int i = 0; i < m; ++i) a[i] *= sig(ld_any(gate, dt, t * gld + (gmode == 1 ? (e + i) / dv : e + i)));
            }
            if (m == 4) { stn<4>(x, dt, base + e, a); return; }
            for (int i = 0; i < m; ++i) st_any(x, dt, base + e + i, a[i]);
          });
}

inline bool al16(const void* q) { return q == nullptr || (reinterpret_cast<uintptr_t>(q) & 15) == 0; }
inline bool rot_vec(int dims, int inter) { return (inter ? dims : dims / 2) % 4 == 0; }

}  // namespace

extern "C" int rb_window_prepare(void* x, int64_t ld, int dt, const void* wq, const void* wk, const float* freq, const float* vfreq, const int* pos,
                                 const int* lens, const int* slots, const int* tok_slot, const int* remain, void* kc, void* vc, int64_t T, int H,
                                 int G, int d, int dv, int dims, int inter, int vdims, int vinter, int keep, int rows, float eps, float mscale, cudaStream_t s) {
  if (T == 0) return 0;
  if (dims % 2 || dims > d || vdims % 2 || vdims > dv || dims / 2 > kMaxHalf || vdims / 2 > kMaxHalf || (pos == nullptr && lens == nullptr)) return -1;
  if ((wq == nullptr) != (wk == nullptr) || (kc == nullptr && vc != nullptr)) return -1;
  PrepareParams p{x, ld, dt, wq, wk, freq, vfreq, pos, lens, slots, tok_slot, remain, kc, vc, H, G, d, dv, dims, inter, vdims, vinter, keep, rows, eps, mscale};
  const bool vec = d % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && rot_vec(dims, inter) && rot_vec(vdims, vinter) && al16(x) && al16(kc) && al16(vc);
  if (wq == nullptr && dims == 0 && vdims == 0) {
    if (kc == nullptr) return 0;
    const bool v4 = d % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && al16(x) && al16(kc) && al16(vc);
    return rb::launch_pdl(v4 ? cache_store_kernel<4> : cache_store_kernel<1>, dim3((unsigned)((T + kThreads / 32 - 1) / (kThreads / 32))), dim3(kThreads), 0, s,
                          p, T) == cudaSuccess ? 0 : 2;
  }
  return rb::launch_pdl(vec ? window_prepare_kernel<4> : window_prepare_kernel<1>, dim3((unsigned)T), dim3(kThreads), 0, s, p) == cudaSuccess ? 0 : 2;
}

extern "C" int rb_turn_gate(void* x, int dt, const void* gate, int64_t gld, int gmode, const float* freq, const int* pos, const int* lens,
                            const int* slots, int64_t T, int H, int dv, int dims, int inter, cudaStream_t s) {
  if (T == 0 || (dims == 0 && gmode == 0)) return 0;
  if (dims % 2 || dims > dv || dims / 2 > kMaxHalf || (pos == nullptr && lens == nullptr)) return -1;
  const bool vec = dv % 4 == 0 && rot_vec(dims, inter) && al16(x) && (gmode != 2 || (gld % 4 == 0 && al16(gate)));
  return rb::launch_pdl(vec ? turn_gate_kernel<4> : turn_gate_kernel<1>, dim3((unsigned)T), dim3(kThreads), 0, s, x, dt, gate, gld, gmode, freq, pos, lens,
                        slots, H, dv, dims, inter) == cudaSuccess ? 0 : 2;
}
