// Kernels between the projections of an attention layer and its attention, in a bf16 and an fp32 build:
//   row norm + store      RMS of q and of k over all heads at once, times weights; q times a factor of its position; k and v
//                         to their pages
//   output gate           attention output times the sigmoid of a projection, heads packed to their true width
//   latent store          latent attention: RMS of the latent (and of the queries' own), rotation of the key part that all
//                         heads share and of the queries' rotated dimensions, page store
//   map store             differential attention: the two maps of a query head as two queries for one key row, page store
//   map difference        differential attention: first map's output minus lambda times the second's, RMS per head, gate
//
// Norms, temperatures, angles and sigmoids are fp32 in both builds.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "launch.cuh"
#include "mixer_util.cuh"

namespace {

using namespace mixer;

template <typename T>
struct Vec {                                               // elements of a 16-byte access
  static constexpr int N = 16 / sizeof(T);
};
template <typename T>
__device__ __forceinline__ void load_vec(const T* p, float (&x)[Vec<T>::N]) {
#pragma unroll
  for (int i = 0; i < Vec<T>::N; i += 4) {
    const float4 v = load4(p + i);
    x[i] = v.x; x[i + 1] = v.y; x[i + 2] = v.z; x[i + 3] = v.w;
  }
}
template <>
__device__ __forceinline__ void load_vec<bf16>(const bf16* p, float (&x)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(h[i]);
    x[2 * i] = f.x;
    x[2 * i + 1] = f.y;
  }
}
__device__ __forceinline__ void store_vec(float* p, const float (&x)[4]) { store4(p, make_float4(x[0], x[1], x[2], x[3])); }
__device__ __forceinline__ void store_vec(bf16* p, const float (&x)[8]) {
  uint4 u;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = u;
}

// two sums over the block at once; `red` holds 66 floats
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
  a = warp_sum(a);
  b = warp_sum(b);
  if ((threadIdx.x & 31) == 0) {
    red[2 * (threadIdx.x >> 5)] = a;
    red[2 * (threadIdx.x >> 5) + 1] = b;
  }
  __syncthreads();
  float2 s = make_float2(0.f, 0.f);
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) {
    s.x += red[2 * w];
    s.y += red[2 * w + 1];
  }
  return s;
}

// ------------------------------------------------------------------------------------------------
// q, k and v of a token at columns 0, off_k, off_v of proj[T, ld].  One CTA per token.  NP > 0: 16-byte pieces, up to NP per
// thread, in registers between norm and store (dim, vdim and all pitches multiples of a piece); NP == 0: any size, read twice.
// ------------------------------------------------------------------------------------------------
struct RowNorm {
  long long ld, num_slots;
  int off_k, off_v, Hq, Hkv, dim, vdim, Dq, Dk, Dv;        // Dq, Dk, Dv: pitches of a head in q_out and in the pages
  int every;                                               // 0: no temperature
  float eps, coef;
};
template <typename T, int NP>
__global__ void __launch_bounds__(512)
row_norm_store_kernel(const T* __restrict__ proj, const int* __restrict__ positions, const int* __restrict__ slots,
                      const float* __restrict__ wq, const float* __restrict__ wk, T* __restrict__ q_out,
                      T* __restrict__ k_cache, T* __restrict__ v_cache, RowNorm p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  __shared__ float red[66];
  const int t = blockIdx.x;
  const T* row = proj + static_cast<size_t>(t) * p.ld;
  const long long slot = slots[t];
  const bool keep = wk != nullptr && slot >= 0 && slot < p.num_slots;     // padding rows have slot -1
  const int nq = p.Hq * p.dim, nk = p.Hkv * p.dim, nv = p.Hkv * p.vdim;
  float temp = 1.f;
  if (p.every > 0) temp = 1.f + p.coef * logf(static_cast<float>((positions[t] + 1) / p.every) + 1.f);
  T* q = q_out + static_cast<size_t>(t) * p.Hq * p.Dq;
  T* k = k_cache + static_cast<size_t>(keep ? slot : 0) * p.Hkv * p.Dk;
  T* v = v_cache + static_cast<size_t>(keep ? slot : 0) * p.Hkv * p.Dv;
  float sq = 0.f, sk = 0.f;
  if constexpr (NP > 0) {
    constexpr int N = Vec<T>::N;
    const int pq = nq / N, pk = keep ? nk / N : 0, pv = keep ? nv / N : 0;
    float x[NP][N];
#pragma unroll
    for (int e = 0; e < NP; ++e) {
      const int i = threadIdx.x + e * blockDim.x;
      if (i < pq + pk + pv) {
        load_vec<T>(i < pq ? row + i * N : i < pq + pk ? row + p.off_k + (i - pq) * N : row + p.off_v + (i - pq - pk) * N, x[e]);
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < N; ++j) s = fmaf(x[e][j], x[e][j], s);
        if (i < pq) sq += s;
        else if (i < pq + pk) sk += s;
      }
    }
    const float2 ss = block_sum2(sq, sk, red);
    const float iq = temp / sqrtf(ss.x / nq + p.eps), ik = 1.f / sqrtf(ss.y / nk + p.eps);
#pragma unroll
    for (int e = 0; e < NP; ++e) {
      const int i = threadIdx.x + e * blockDim.x;
      if (i >= pq + pk + pv) continue;
      T* dst;
      if (i < pq + pk) {
        const bool is_q = i < pq;
        const int c = (is_q ? i : i - pq) * N, h = c / p.dim, pitch = is_q ? p.Dq : p.Dk;
        const float* w = (is_q ? wq : wk) + c;
        const float inv = is_q ? iq : ik;
#pragma unroll
        for (int j = 0; j < N; j += 4) {
          const float4 f = *reinterpret_cast<const float4*>(w + j);
          x[e][j] *= inv * f.x; x[e][j + 1] *= inv * f.y; x[e][j + 2] *= inv * f.z; x[e][j + 3] *= inv * f.w;
        }
        dst = (is_q ? q : k) + static_cast<size_t>(h) * pitch + (c - h * p.dim);
      } else {
        const int c = (i - pq - pk) * N, h = c / p.vdim;
        dst = v + static_cast<size_t>(h) * p.Dv + (c - h * p.vdim);
      }
      store_vec(dst, x[e]);
    }
  } else {
    for (int i = threadIdx.x; i < nq; i += blockDim.x) sq += to_f(row[i]) * to_f(row[i]);
    if (keep)
      for (int i = threadIdx.x; i < nk; i += blockDim.x) sk += to_f(row[p.off_k + i]) * to_f(row[p.off_k + i]);
    const float2 ss = block_sum2(sq, sk, red);
    const float iq = temp / sqrtf(ss.x / nq + p.eps), ik = 1.f / sqrtf(ss.y / nk + p.eps);
    for (int i = threadIdx.x; i < nq; i += blockDim.x) put(q + i / p.dim * p.Dq + i % p.dim, to_f(row[i]) * iq * wq[i]);
    if (keep) {
      for (int i = threadIdx.x; i < nk; i += blockDim.x) put(k + i / p.dim * p.Dk + i % p.dim, to_f(row[p.off_k + i]) * ik * wk[i]);
      for (int i = threadIdx.x; i < nv; i += blockDim.x) v[i / p.vdim * p.Dv + i % p.vdim] = row[p.off_v + i];
    }
  }
  const int pad = p.Dq - p.dim;
  if (pad > 0)
    for (int i = threadIdx.x; i < p.Hq * pad; i += blockDim.x) put(q + i / pad * p.Dq + p.dim + i % pad, 0.f);
}

// ------------------------------------------------------------------------------------------------
// out[t, h * width + i] = x[t, h, i] * sigmoid(gate[t, h * width + i]); x has heads `pitch` elements apart
// ------------------------------------------------------------------------------------------------
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
output_gate_kernel(const T* __restrict__ x, const T* __restrict__ gate, long long ld, T* __restrict__ out, long long n, int H,
                   int pitch, int width) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  constexpr int N = VEC ? Vec<T>::N : 1;
  const long long stride = static_cast<long long>(gridDim.x) * blockDim.x;
  const unsigned cols = static_cast<unsigned>(H * width);
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n / N; i += stride) {
    const long long e = i * N, t = e / cols;
    const unsigned c = static_cast<unsigned>(e - t * cols), h = c / width;
    const T* src = x + (t * H + h) * pitch + (c - h * width);
    const T* g = gate + t * ld + c;
    if constexpr (VEC) {
      float a[N], b[N];
      load_vec<T>(src, a);
      load_vec<T>(g, b);
#pragma unroll
      for (int j = 0; j < N; ++j) a[j] *= sigmoid_t<T>(b[j]);
      store_vec(out + e, a);
    } else {
      put(out + e, to_f(*src) * sigmoid_t<T>(to_f(*g)));
    }
  }
}

// ------------------------------------------------------------------------------------------------
// Inputs of latent attention.  proj[T, ld]: latent (rank) and the shared key's rotated part (rot) at off_c; q[T, ld_q]: queries
// (H heads of dim plain and rot rotated dimensions).  Grid (T, groups): the first warp normalises the latent and rotates the
// shared part (pages null: not wanted), the second normalises the queries' latent (cq_rank columns at off_cq, to
// cq_out[T, ld_cq], zeros behind them; null: not wanted), all rotate the queries of a head each.  Pairs 2i, 2i + 1.  Rotated
// dimensions go to q_out from column off_rot on (null: not wanted), whole queries (plain, rotated, zeros) to q_full, `full`
// columns per head (null: not wanted).  VEC: every offset, size and pitch is a multiple of 8 elements; a lane then takes 8 at a time.
// ------------------------------------------------------------------------------------------------
struct Latent {
  long long ld, num_slots;
  int off_c, rank, rot, H, dim, off_rot, width, max_pos;   // width: of a cached row and of a head of q_out
  int full;
  float eps;
  long long ld_q;
  int off_cq, cq_rank, ld_cq;
};
template <typename T>
__device__ __forceinline__ void load8(const T* p, float (&x)[8]) {
  if constexpr (sizeof(T) == 2) {
    load_vec<T>(p, x);
  } else {
    const float4 a = load4(p), b = load4(p + 4);
    x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w;
    x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
  }
}
template <typename T>
__device__ __forceinline__ void store8(T* p, const float (&x)[8]) {
  if constexpr (sizeof(T) == 2) {
    store_vec(p, x);
  } else {
    store4(p, make_float4(x[0], x[1], x[2], x[3]));
    store4(p + 4, make_float4(x[4], x[5], x[6], x[7]));
  }
}
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
latent_store_kernel(const T* __restrict__ proj, const float* __restrict__ weight, const int* __restrict__ positions,
                    const float* __restrict__ cos_sin, const int* __restrict__ slots, T* __restrict__ pages,
                    const T* __restrict__ q_in, T* __restrict__ q_out, T* __restrict__ q_full,
                    const float* __restrict__ cq_weight, T* __restrict__ cq_out, Latent p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warps = (blockDim.x >> 5) * gridDim.y;
  const int warp = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const T* row = proj + static_cast<size_t>(t) * p.ld;
  const int rh = p.rot / 2, pos = min(max(positions[t], 0), p.max_pos - 1);
  const float* cs = cos_sin + static_cast<size_t>(pos) * p.rot;
  const float zero[8] = {};
  auto rotate = [&](const T* src, T* dst, int end, int l, int step) {      // rotated pairs, then zeros up to `end`
    if constexpr (VEC) {
      for (int i = 8 * l; i < end; i += 8 * step) {
        if (i >= p.rot) {
          store8(dst + i, zero);
          continue;
        }
        float x[8];
        load8(src + i, x);
        const float4 c = *reinterpret_cast<const float4*>(cs + i / 2), s = *reinterpret_cast<const float4*>(cs + rh + i / 2);
        const float y[8] = {x[0] * c.x - x[1] * s.x, x[1] * c.x + x[0] * s.x, x[2] * c.y - x[3] * s.y, x[3] * c.y + x[2] * s.y,
                            x[4] * c.z - x[5] * s.z, x[5] * c.z + x[4] * s.z, x[6] * c.w - x[7] * s.w, x[7] * c.w + x[6] * s.w};
        store8(dst + i, y);
      }
    } else {
      for (int i = l; i < rh; i += step) {
        const float u = to_f(src[2 * i]), v = to_f(src[2 * i + 1]), c = cs[i], s = cs[rh + i];
        put(dst + 2 * i, u * c - v * s);
        put(dst + 2 * i + 1, v * c + u * s);
      }
      for (int i = p.rot + l; i < end; i += step) put(dst + i, 0.f);
    }
  };
  // c over its root mean square times w
  auto norm_row = [&](const T* c, const float* w, T* dst, int n) {
    float ss = 0.f;
    if constexpr (VEC) {
      constexpr int kHeld = 2;                             // pieces per lane that stay in registers
      float x[kHeld][8];
#pragma unroll
      for (int e = 0; e < kHeld; ++e) {
        const int i = 8 * (lane + 32 * e);
#pragma unroll
        for (int k = 0; k < 8; ++k) x[e][k] = 0.f;
        if (i < n) load8(c + i, x[e]);
#pragma unroll
        for (int k = 0; k < 8; ++k) ss = fmaf(x[e][k], x[e][k], ss);
      }
      for (int i = 8 * (lane + 32 * kHeld); i < n; i += 256) {
        float y[8];
        load8(c + i, y);
#pragma unroll
        for (int k = 0; k < 8; ++k) ss = fmaf(y[k], y[k], ss);
      }
      const float inv = 1.f / sqrtf(warp_sum(ss) / n + p.eps);
      auto emit = [&](int i, float (&y)[8]) {
#pragma unroll
        for (int k = 0; k < 8; k += 4) {
          const float4 f = *reinterpret_cast<const float4*>(w + i + k);
          y[k] *= inv * f.x; y[k + 1] *= inv * f.y; y[k + 2] *= inv * f.z; y[k + 3] *= inv * f.w;
        }
        store8(dst + i, y);
      };
#pragma unroll
      for (int e = 0; e < kHeld; ++e) {
        const int i = 8 * (lane + 32 * e);
        if (i < n) emit(i, x[e]);
      }
      for (int i = 8 * (lane + 32 * kHeld); i < n; i += 256) {
        float y[8];
        load8(c + i, y);
        emit(i, y);
      }
    } else {
      for (int i = lane; i < n; i += 32) ss = fmaf(to_f(c[i]), to_f(c[i]), ss);
      const float inv = 1.f / sqrtf(warp_sum(ss) / n + p.eps);
      for (int i = lane; i < n; i += 32) put(dst + i, to_f(c[i]) * inv * w[i]);
    }
  };
  if (warp == 0 && pages != nullptr) {
    const long long slot = slots[t];
    if (slot >= 0 && slot < p.num_slots) {                 // padding rows have slot -1
      const T* c = row + p.off_c;
      T* dst = pages + static_cast<size_t>(slot) * p.width;
      norm_row(c, weight, dst, p.rank);
      if (p.rot > 0) rotate(c + p.rank, dst + p.off_rot, p.rot, lane, 32);
    }
  }
  if (warp == warps - 1 && cq_out != nullptr) {
    T* dst = cq_out + static_cast<size_t>(t) * p.ld_cq;
    norm_row(row + p.off_cq, cq_weight, dst, p.cq_rank);
    for (int i = p.cq_rank + lane; i < p.ld_cq; i += 32) put(dst + i, 0.f);
  }
  if (q_in == nullptr) return;
  // eight lanes per head
  const int l = lane & 7, tail = p.width - p.off_rot;
  for (int h = 4 * warp + (lane >> 3); h < p.H; h += 4 * warps) {
    const T* q = q_in + static_cast<size_t>(t) * p.ld_q + static_cast<size_t>(h) * (p.dim + p.rot);
    if (q_out != nullptr && tail > 0) rotate(q + p.dim, q_out + (static_cast<size_t>(t) * p.H + h) * p.width + p.off_rot, tail, l, 8);
    if (q_full != nullptr) {
      T* dst = q_full + (static_cast<size_t>(t) * p.H + h) * p.full;
      if constexpr (VEC) {
        for (int i = 8 * l; i < p.dim; i += 64) {
          float x[8];
          load8(q + i, x);
          store8(dst + i, x);
        }
      } else {
        for (int i = l; i < p.dim; i += 8) dst[i] = q[i];
      }
      rotate(q + p.dim, dst + p.dim, p.full - p.dim, l, 8);
    }
  }
}

// ------------------------------------------------------------------------------------------------
// Inputs of differential attention.  proj[T, ld]: q (H heads of two maps of `dim`) at column 0, k (G heads, two maps of `dim`)
// at off_k, v (G of vdim) at off_v.  A key row in the pages holds both maps of a head side by side (2 dim of Dk columns), and
// every query map becomes a query of its own for that row: zeros but for its own half, q_out[T, 2 H, Dk].  So one attention
// over G key heads reads keys and values once for both maps.  One CTA per token; VEC: 16-byte pieces.
// ------------------------------------------------------------------------------------------------
struct Maps {
  long long ld, num_slots;
  int off_k, off_v, H, G, dim, vdim, Dk, Dv;               // Dk, Dv: pitches of a head in q_out and in the pages
};
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
map_store_kernel(const T* __restrict__ proj, const int* __restrict__ slots, T* __restrict__ q_out, T* __restrict__ k_cache,
                 T* __restrict__ v_cache, Maps p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  constexpr int N = VEC ? Vec<T>::N : 1;
  const int t = blockIdx.x;
  const T* row = proj + static_cast<size_t>(t) * p.ld;
  const long long slot = slots[t];
  const bool keep = slot >= 0 && slot < p.num_slots;       // padding rows have slot -1
  auto copy = [&](T* dst, const T* src) {
    if constexpr (VEC) *reinterpret_cast<uint4*>(dst) = src != nullptr ? *reinterpret_cast<const uint4*>(src) : make_uint4(0, 0, 0, 0);
    else *dst = src != nullptr ? *src : T(0.f);
  };
  const int per = p.Dk / N, nq = 2 * p.H * per, nk = keep ? p.G * 2 * p.dim / N : 0, nv = keep ? p.G * p.vdim / N : 0;
  T* q = q_out + static_cast<size_t>(t) * 2 * p.H * p.Dk;
  for (int i = threadIdx.x; i < nq + nk + nv; i += blockDim.x) {
    if (i < nq) {
      const int h = i / per, c = (i - h * per) * N, at = c - (h & 1) * p.dim;
      copy(q + static_cast<size_t>(h) * p.Dk + c, at >= 0 && at < p.dim ? row + static_cast<size_t>(h) * p.dim + at : nullptr);
    } else if (i < nq + nk) {
      const int c = (i - nq) * N, g = c / (2 * p.dim);
      copy(k_cache + (static_cast<size_t>(slot) * p.G + g) * p.Dk + (c - g * 2 * p.dim), row + p.off_k + c);
    } else {
      const int c = (i - nq - nk) * N, g = c / p.vdim;
      copy(v_cache + (static_cast<size_t>(slot) * p.G + g) * p.Dv + (c - g * p.vdim), row + p.off_v + c);
    }
  }
}

// out[t, h] = (a[t, 2h] - lambda a[t, 2h + 1]) over its root mean square (vdim values, plus eps), times `factor` and the sigmoid
// of gate[t, h] (null: none).  a has heads `pitch` elements apart; out rows are H * vdim wide.  L lanes per (token, head), a
// piece of E elements at a time, NP pieces per lane; NP 0: any size, read twice.
template <typename T, int L, int E, int NP>
__global__ void __launch_bounds__(256)
map_difference_kernel(const T* __restrict__ a, const T* __restrict__ gate, long long ld_gate, T* __restrict__ out, long long jobs,
                      int H, int pitch, int vdim, float lambda, float factor, float eps) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int l = threadIdx.x % L;
  const long long job = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) / L;
  const bool on = job < jobs;                              // lanes past the last head stay for the exchanges
  const long long at = on ? job : jobs - 1, t = at / H, h = at - t * H;
  const T* x = a + static_cast<size_t>(at) * 2 * pitch;
  const T* y = x + pitch;
  T* dst = out + static_cast<size_t>(at) * vdim;
  auto load = [&](int i, float (&d)[E]) {
    if constexpr (E == Vec<T>::N) {
      float u[E], v[E];
      load_vec<T>(x + i, u);
      load_vec<T>(y + i, v);
#pragma unroll
      for (int k = 0; k < E; ++k) d[k] = fmaf(-lambda, v[k], u[k]);
    } else {
#pragma unroll
      for (int k = 0; k < E; ++k) d[k] = fmaf(-lambda, to_f(y[i + k]), to_f(x[i + k]));
    }
  };
  float ss = 0.f, d[NP > 0 ? NP : 1][E];
  if constexpr (NP > 0) {
#pragma unroll
    for (int e = 0; e < NP; ++e) {
      const int i = (l + e * L) * E;
      if (i < vdim) {
        load(i, d[e]);
#pragma unroll
        for (int k = 0; k < E; ++k) ss = fmaf(d[e][k], d[e][k], ss);
      }
    }
  } else {
    for (int i = l * E; i < vdim; i += L * E) {
      load(i, d[0]);
#pragma unroll
      for (int k = 0; k < E; ++k) ss = fmaf(d[0][k], d[0][k], ss);
    }
  }
#pragma unroll
  for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!on) return;
  float f = factor / sqrtf(ss / vdim + eps);
  if (gate != nullptr) f *= sigmoid_t<T>(to_f(gate[t * ld_gate + h]));
  auto emit = [&](int i, float (&v)[E]) {
#pragma unroll
    for (int k = 0; k < E; ++k) v[k] *= f;
    if constexpr (E == Vec<T>::N) {
      store_vec(dst + i, v);
    } else {
#pragma unroll
      for (int k = 0; k < E; ++k) put(dst + i + k, v[k]);
    }
  };
  if constexpr (NP > 0) {
#pragma unroll
    for (int e = 0; e < NP; ++e) {
      const int i = (l + e * L) * E;
      if (i < vdim) emit(i, d[e]);
    }
  } else {
    for (int i = l * E; i < vdim; i += L * E) {
      load(i, d[0]);
      emit(i, d[0]);
    }
  }
}

int done() { return cudaGetLastError() == cudaSuccess ? 0 : -3; }

template <typename T>
int row_norm_store(const void* proj, const int* positions, const int* slots, const float* wq, const float* wk, void* q_out,
                   void* k_cache, void* v_cache, int T_, const RowNorm& p, cudaStream_t stream) {
  constexpr int N = Vec<T>::N;
  auto go = [&](auto kern, int threads) {
    tgi::launch(kern, dim3(T_), dim3(threads), 0, stream, static_cast<const T*>(proj), positions, slots, wq, wk,
                static_cast<T*>(q_out), static_cast<T*>(k_cache), static_cast<T*>(v_cache), p);
    return done();
  };
  const int pieces = (p.Hq * p.dim + (wk != nullptr ? p.Hkv * (p.dim + p.vdim) : 0)) / N;
  const bool vec = p.dim % N == 0 && p.vdim % N == 0 && p.Dq % N == 0 && p.Dk % N == 0 && p.Dv % N == 0 && p.ld % N == 0 &&
                   p.off_k % N == 0 && p.off_v % N == 0 && reinterpret_cast<uintptr_t>(proj) % 16 == 0;
  if (vec && pieces <= 4 * 512) {
    const int threads = pieces >= 1024 ? 512 : pieces >= 256 ? 256 : 128;
    const int np = (pieces + threads - 1) / threads;
    return np <= 1 ? go(row_norm_store_kernel<T, 1>, threads) : np <= 2 ? go(row_norm_store_kernel<T, 2>, threads)
                                                                       : go(row_norm_store_kernel<T, 4>, threads);
  }
  return go(row_norm_store_kernel<T, 0>, 256);
}

template <typename T>
int output_gate(const void* x, const void* gate, long long ld, void* out, int T_, int H, int pitch, int width, cudaStream_t stream) {
  constexpr int N = Vec<T>::N;
  const bool vec = width % N == 0 && pitch % N == 0 && ld % N == 0 && reinterpret_cast<uintptr_t>(gate) % 16 == 0;
  const long long n = static_cast<long long>(T_) * H * width;
  long long blocks = (n / (vec ? N : 1) + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  auto go = [&](auto kern) {
    tgi::launch(kern, dim3(static_cast<unsigned>(blocks)), dim3(256), 0, stream, static_cast<const T*>(x),
                static_cast<const T*>(gate), ld, static_cast<T*>(out), n, H, pitch, width);
    return done();
  };
  return vec ? go(output_gate_kernel<T, true>) : go(output_gate_kernel<T, false>);
}

template <typename T>
int map_store(const void* proj, const int* slots, void* q_out, void* k_cache, void* v_cache, int T_, const Maps& p,
              cudaStream_t stream) {
  constexpr int N = Vec<T>::N;
  const bool vec = p.dim % N == 0 && p.vdim % N == 0 && p.Dk % N == 0 && p.Dv % N == 0 && p.ld % N == 0 && p.off_k % N == 0 &&
                   p.off_v % N == 0 && reinterpret_cast<uintptr_t>(proj) % 16 == 0;
  auto go = [&](auto kern) {
    tgi::launch(kern, dim3(T_), dim3(256), 0, stream, static_cast<const T*>(proj), slots, static_cast<T*>(q_out),
                static_cast<T*>(k_cache), static_cast<T*>(v_cache), p);
    return done();
  };
  return vec ? go(map_store_kernel<T, true>) : go(map_store_kernel<T, false>);
}

template <typename T>
int map_difference(const void* a, const void* gate, long long ld_gate, void* out, int T_, int H, int pitch, int vdim, float lambda,
                   float factor, float eps, cudaStream_t stream) {
  constexpr int N = Vec<T>::N;
  const long long jobs = static_cast<long long>(T_) * H;
  auto go = [&](auto kern, int lanes) {
    tgi::launch(kern, dim3(static_cast<unsigned>((jobs * lanes + 255) / 256)), dim3(256), 0, stream, static_cast<const T*>(a),
                static_cast<const T*>(gate), ld_gate, static_cast<T*>(out), jobs, H, pitch, vdim, lambda, factor, eps);
    return done();
  };
  if (vdim % N == 0 && pitch % N == 0) {
    const int pieces = vdim / N;
    if (pieces <= 16) return go(map_difference_kernel<T, 16, N, 1>, 16);
    if (pieces <= 32) return go(map_difference_kernel<T, 32, N, 1>, 32);
    return go(map_difference_kernel<T, 32, N, 0>, 32);
  }
  return go(map_difference_kernel<T, 32, 1, 0>, 32);
}

}  // namespace

// `f32` selects the build: 1 = fp32 activations and pages, 0 = bf16.
extern "C" {

// wk null: the layer has queries only and nothing is stored.  every 0: no temperature.
int tgi_row_norm_store(int f32, const void* proj, long long ld, int off_k, int off_v, const int* positions, const int* slots,
                       const float* wq, const float* wk, void* q_out, void* k_cache, void* v_cache, int T, int Hq, int Hkv,
                       int dim, int vdim, int Dq, int Dk, int Dv, long long num_slots, float eps, float coef, int every,
                       cudaStream_t stream) {
  if (T <= 0) return 0;
  if (Dq < dim || Dk < dim || Dv < vdim || every < 0) return -10;
  const RowNorm p{ld, num_slots, off_k, off_v, Hq, Hkv, dim, vdim, Dq, Dk, Dv, every, eps, coef};
  return f32 ? row_norm_store<float>(proj, positions, slots, wq, wk, q_out, k_cache, v_cache, T, p, stream)
             : row_norm_store<bf16>(proj, positions, slots, wq, wk, q_out, k_cache, v_cache, T, p, stream);
}

int tgi_output_gate(int f32, const void* x, const void* gate, long long ld, void* out, int T, int H, int pitch, int width,
                    cudaStream_t stream) {
  if (T <= 0) return 0;
  if (pitch < width || width < 1) return -10;
  return f32 ? output_gate<float>(x, gate, ld, out, T, H, pitch, width, stream)
             : output_gate<bf16>(x, gate, ld, out, T, H, pitch, width, stream);
}

// pages null: no latent is stored (proj may be null).  q null: no queries.  cq_out null: no latent of queries.
int tgi_latent_store(int f32, const void* proj, long long ld, int off_c, const float* weight, float eps, const int* positions,
                     const float* cos_sin, int max_pos, const int* slots, void* pages, long long num_slots, const void* q,
                     long long ld_q, void* q_out, void* q_full, int off_cq, int cq_rank, const float* cq_weight, void* cq_out,
                     int ld_cq, int T, int H, int dim, int rank, int rot, int off_rot, int width, int full, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (rot % 2 != 0 || off_rot < rank || width < off_rot + rot || max_pos < 1 || (q_full != nullptr && full < dim + rot) ||
      (cq_out != nullptr && ld_cq < cq_rank))
    return -10;
  const Latent p{ld, num_slots, off_c, rank, rot, H, dim, off_rot, width, max_pos, full, eps, ld_q, off_cq, cq_rank, ld_cq};
  const bool heads = q != nullptr && (q_full != nullptr || (q_out != nullptr && width > off_rot));
  const int least = cq_out != nullptr && pages != nullptr ? 2 : 1;
  int want = heads ? (H + 3) / 4 : 1;                      // four heads per warp at a time
  want = want < least ? least : want;
  const int warps = want < 4 ? want : 4;
  const int groups = T >= 1024 ? 1 : (want + warps - 1) / warps;
  auto aligned = [](const void* x) { return reinterpret_cast<uintptr_t>(x) % 16 == 0; };
  const bool vec = dim % 8 == 0 && rot % 8 == 0 && rank % 8 == 0 && off_c % 8 == 0 && ld % 8 == 0 && off_rot % 8 == 0 && width % 8 == 0 &&
                   (q_full == nullptr || full % 8 == 0) && aligned(proj) && (q == nullptr || (ld_q % 8 == 0 && aligned(q))) &&
                   (cq_out == nullptr || (off_cq % 8 == 0 && cq_rank % 8 == 0 && ld_cq % 8 == 0));
  auto go = [&](auto kern, auto tag) {
    using E = decltype(tag);
    tgi::launch(kern, dim3(T, groups), dim3(32 * warps), 0, stream, static_cast<const E*>(proj), weight, positions, cos_sin, slots,
                static_cast<E*>(pages), static_cast<const E*>(q), static_cast<E*>(q_out), static_cast<E*>(q_full), cq_weight,
                static_cast<E*>(cq_out), p);
    return done();
  };
  if (vec) return f32 ? go(latent_store_kernel<float, true>, float()) : go(latent_store_kernel<bf16, true>, bf16());
  return f32 ? go(latent_store_kernel<float, false>, float()) : go(latent_store_kernel<bf16, false>, bf16());
}

int tgi_map_store(int f32, const void* proj, long long ld, int off_k, int off_v, const int* slots, void* q_out, void* k_cache,
                  void* v_cache, int T, int H, int G, int dim, int vdim, int Dk, int Dv, long long num_slots, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (Dk < 2 * dim || Dv < vdim || dim < 1) return -10;
  const Maps p{ld, num_slots, off_k, off_v, H, G, dim, vdim, Dk, Dv};
  return f32 ? map_store<float>(proj, slots, q_out, k_cache, v_cache, T, p, stream)
             : map_store<bf16>(proj, slots, q_out, k_cache, v_cache, T, p, stream);
}

int tgi_map_difference(int f32, const void* a, const void* gate, long long ld_gate, void* out, int T, int H, int pitch, int vdim,
                       float lambda, float factor, float eps, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (pitch < vdim || vdim < 1 || H < 1) return -10;
  return f32 ? map_difference<float>(a, gate, ld_gate, out, T, H, pitch, vdim, lambda, factor, eps, stream)
             : map_difference<bf16>(a, gate, ld_gate, out, T, H, pitch, vdim, lambda, factor, eps, stream);
}

}  // extern "C"
