// Recurrent token mixers with a matrix state per head, S[dim x vdim] in fp32:
//
//   gated delta rule, one decay per key channel      S <- g * S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   linear attention with a fixed decay per head     S <- d S + k v^T;                                    o = S^T q
//
// The columns of S never meet: column j of a head needs k, q, g of the head and only v_j of its own.
//
// scan_kernel walks the tokens a sequence brings in this step with the state in registers (one load and one store of
// the state per step, whatever the number of tokens).  Sixteen lanes share CN columns, lane l holding rows
// 4 l + 64 j + (0..3) of each: a 16-byte shared-memory read of k (q, g) then feeds 4 CN multiply-adds, done in pairs
// (fma.rn.f32x2).  The sums of the CN columns are reduced by halving exchanges, after which every lane owns one
// column; the lane of a column forms its u and read-out.  Tiles of kTile tokens are staged in shared memory one tile
// ahead.  For the delta rule the tile also holds g * k and g * q, because
//   S_new^T q = (g S)^T q + (k . q) u = S^T (g q) + (k . q) u
// lets both dot products run on the old state: one reduction per token sits on the critical path, not two.
// step_kernel is the single-token form of decode: eight lanes per column, no staging, bound by reading and writing the
// state once.
//
// Pools are [slots, H, vdim, dimP] with dimP = dim rounded up to 32; rows dim .. dimP - 1 stay zero.  A sequence whose
// step starts at position 0 starts from a zero state without reading its slot; slot -1 (padding rows of a captured
// batch) reads and writes nothing.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "launch.cuh"

namespace {

using bf16 = __nv_bfloat16;
constexpr int kTile = 8;          // tokens per staged tile
constexpr int kThreads = 128;

__device__ __forceinline__ float to_f(float x) { return x; }
__device__ __forceinline__ float to_f(bf16 x) { return __bfloat162float(x); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }

struct ScanArgs {
  // delta rule: fp32 q, k [T, G, dimP], g [T, H, dimP], v [T, H, vdim], beta [T, H], qk = q . k [T, G]
  const float *q, *k, *g, *v, *beta, *qk;
  // linear attention: proj [T, ld] with q, k (H x dim) and v (H x vdim) at off_q, off_k, off_v (SiLU applied here)
  const void* proj;
  long long ld;
  int off_q, off_k, off_v;
  const float* decay;             // [H]
  const int* cu;                  // [B + 1]
  const int* kv_lens;             // [B] tokens of the sequence including this step's
  const int* state_slots;         // [B]
  float* state;                   // [num_slots, H, vdim, dimP]
  float* out;                     // [T, H, vdim]
  int num_slots, G, H, dim, dimP, vdim;
  int vec;                        // proj: heads may be read four elements at a time
};

// sum over the eight lanes of a column group
__device__ __forceinline__ float sum8(float v) {
  v += __shfl_xor_sync(0xffffffffu, v, 1);
  v += __shfl_xor_sync(0xffffffffu, v, 2);
  v += __shfl_xor_sync(0xffffffffu, v, 4);
  return v;
}

// two fp32 in a 64-bit register
using pair = unsigned long long;
__device__ __forceinline__ pair pk(float x, float y) {
  pair r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
  return r;
}
__device__ __forceinline__ float pair_sum(pair p) {
  float x, y;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(p));
  return x + y;
}
__device__ __forceinline__ pair fma2(pair a, pair b, pair c) {
  pair r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ pair mul2(pair a, pair b) {
  pair r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// Sums of CN values over sixteen lanes; lane l ends with the total of value l / (16 / CN).
template <int CN>
__device__ __forceinline__ float scatter_sum(float (&v)[CN], int l) {
  int m = 8;
#pragma unroll
  for (int half = CN / 2; half >= 1; half /= 2, m >>= 1) {
    const bool up = l & m;
#pragma unroll
    for (int i = 0; i < half; ++i) {
      const float give = up ? v[i] : v[i + half], keep = up ? v[i + half] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, m);
    }
  }
#pragma unroll
  for (; m >= 1; m >>= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], m);
  return v[0];
}

__device__ __forceinline__ float4 raw4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 raw4(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
// columns c .. c + 3 of a head after SiLU, zero past `dim`; `vec`: the four may be read at once
template <typename T>
__device__ __forceinline__ float4 load4_silu(const T* p, int c, int dim, bool vec) {
  if (vec && c < dim) {
    const float4 x = raw4(p + c);
    return make_float4(silu_f(x.x), silu_f(x.y), silu_f(x.z), silu_f(x.w));
  }
  float v[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) v[i] = c + i < dim ? silu_f(to_f(p[c + i])) : 0.f;
  return make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }

template <bool DELTA, int J, int CN>
struct ScanSmem {
  static constexpr int kRow = 64 * J;
  static constexpr int kCols = 8 * CN;                          // columns of a CTA
  static constexpr int kArrays = DELTA ? 4 : 2;                 // k, g, g k, g q   |   k, q
  static constexpr int kVec = kTile * kRow;                     // floats of one array
  static constexpr int kStage = kArrays * kVec + kTile * kCols + 2 * kTile;   // + v tile, beta, q . k
  static constexpr int kBytes = 2 * kStage * 4;
};

// grid (ceil(vdim / (8 CN)), H, B), 128 threads: eight groups of sixteen lanes, CN columns per group
template <typename T, bool DELTA, int J, int CN>
__global__ void __launch_bounds__(kThreads)
scan_kernel(ScanArgs p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  extern __shared__ __align__(16) float smem[];
  using S = ScanSmem<DELTA, J, CN>;
  constexpr int NI = J;                                         // float4 pieces per thread of one array: kTile 16 J / 128
  constexpr int NV = kTile * S::kCols / kThreads;
  static_assert(kTile * 16 == kThreads, "a tile row is 16 J pieces");
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * S::kCols;
  const int begin = p.cu[b], n = p.cu[b + 1] - begin;
  if (n <= 0) return;
  const int start = p.kv_lens[b] - n, slot = p.state_slots[b];
  const bool has = slot >= 0 && slot < p.num_slots;
  const int tid = threadIdx.x, l = tid & 15;
  const int col = (tid >> 4) * CN;                              // first column of this group, inside the tile
  const int mine = l / (16 / CN);                               // the column whose sums this lane ends up with
  const int hg = h / (p.H / p.G);
  float* st0 = p.state + ((static_cast<size_t>(has ? slot : 0) * p.H + h) * p.vdim + c0 + col) * p.dimP + 4 * l;
  const bool store_out = l % (16 / CN) == 0 && c0 + col + mine < p.vdim;

  pair s[CN][J][2];
#pragma unroll
  for (int c = 0; c < CN; ++c) {
#pragma unroll
    for (int j = 0; j < J; ++j) {
      s[c][j][0] = s[c][j][1] = 0ull;
      if (has && start > 0 && c0 + col + c < p.vdim && 4 * l + 64 * j < p.dimP) {
        const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(st0 + c * p.dimP + 64 * j);
        s[c][j][0] = v.x;
        s[c][j][1] = v.y;
      }
    }
  }

  float4 rk[NI], rq[NI], rg[DELTA ? NI : 1];
  float rv[NV], rb = 0.f, rd = 0.f;
  auto fetch = [&](int t0) {                                    // tokens t0 .. of the sequence into registers
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int it = tid + i * kThreads, tk = it / (16 * J), c4 = (it % (16 * J)) * 4;
      const bool ok = t0 + tk < n && c4 < p.dimP;
      const size_t t = begin + t0 + tk;
      const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
      if (DELTA) {
        rk[i] = ok ? raw4(p.k + (t * p.G + hg) * p.dimP + c4) : z;
        rq[i] = ok ? raw4(p.q + (t * p.G + hg) * p.dimP + c4) : z;
        rg[DELTA ? i : 0] = ok ? raw4(p.g + (t * p.H + h) * p.dimP + c4) : z;
      } else {
        const T* row = static_cast<const T*>(p.proj) + t * p.ld + h * p.dim;
        rk[i] = ok ? load4_silu(row + p.off_k, c4, p.dim, p.vec) : z;
        rq[i] = ok ? load4_silu(row + p.off_q, c4, p.dim, p.vec) : z;
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int it = tid + i * kThreads, tk = it / S::kCols, c = c0 + it % S::kCols;
      const bool ok = t0 + tk < n && c < p.vdim;
      const size_t t = begin + t0 + tk;
      if (DELTA) rv[i] = ok ? p.v[(t * p.H + h) * p.vdim + c] : 0.f;
      else rv[i] = ok ? silu_f(to_f(static_cast<const T*>(p.proj)[t * p.ld + p.off_v + h * p.vdim + c])) : 0.f;
    }
    if (DELTA && tid < kTile) {
      const bool ok = t0 + tid < n;
      const size_t t = begin + t0 + tid;
      rb = ok ? p.beta[t * p.H + h] : 0.f;
      rd = ok ? p.qk[t * p.G + hg] : 0.f;
    }
  };
  auto stage = [&](float* d) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      float4* k4 = reinterpret_cast<float4*>(d) + tid + i * kThreads;
      k4[0] = rk[i];
      if (DELTA) {
        k4[S::kVec / 4] = rg[DELTA ? i : 0];
        k4[2 * (S::kVec / 4)] = mul4(rg[DELTA ? i : 0], rk[i]);
        k4[3 * (S::kVec / 4)] = mul4(rg[DELTA ? i : 0], rq[i]);
      } else {
        k4[S::kVec / 4] = rq[i];
      }
    }
    float* v = d + S::kArrays * S::kVec;
#pragma unroll
    for (int i = 0; i < NV; ++i) v[tid + i * kThreads] = rv[i];
    if (DELTA && tid < kTile) {
      v[kTile * S::kCols + tid] = rb;
      v[kTile * S::kCols + kTile + tid] = rd;
    }
  };
  const float dec = DELTA ? 0.f : p.decay[h];
  const pair dec2 = pk(dec, dec);
  fetch(0);
  stage(smem);
  __syncthreads();
  float* const out0 = p.out + (static_cast<size_t>(begin) * p.H + h) * p.vdim + c0 + col + mine;
  const size_t out_step = static_cast<size_t>(p.H) * p.vdim;
  for (int t0 = 0, cur = 0; t0 < n; t0 += kTile, cur ^= 1) {
    const bool more = t0 + kTile < n;
    if (more) fetch(t0 + kTile);
    const float* d = smem + cur * S::kStage;
    const float* vt = d + S::kArrays * S::kVec;
    const int cnt = min(kTile, n - t0);
#pragma unroll 1
    for (int i = 0; i < cnt; ++i) {
      const float* kr = d + i * S::kRow + 4 * l;
      float o;
      if (DELTA) {
        pair a2[CN], w2[CN];
#pragma unroll
        for (int c = 0; c < CN; ++c) a2[c] = w2[c] = 0ull;
#pragma unroll
        for (int j = 0; j < J; ++j) {
          const ulonglong2 gk = *reinterpret_cast<const ulonglong2*>(kr + 2 * S::kVec + 64 * j);
          const ulonglong2 gq = *reinterpret_cast<const ulonglong2*>(kr + 3 * S::kVec + 64 * j);
#pragma unroll
          for (int c = 0; c < CN; ++c) a2[c] = fma2(s[c][j][1], gk.y, fma2(s[c][j][0], gk.x, a2[c]));
#pragma unroll
          for (int c = 0; c < CN; ++c) w2[c] = fma2(s[c][j][1], gq.y, fma2(s[c][j][0], gq.x, w2[c]));
        }
        float a[CN], w[CN];
#pragma unroll
        for (int c = 0; c < CN; ++c) {
          a[c] = pair_sum(a2[c]);
          w[c] = pair_sum(w2[c]);
        }
        const float beta = vt[kTile * S::kCols + i], kq = vt[kTile * S::kCols + kTile + i];
        const float u = beta * (vt[i * S::kCols + col + mine] - scatter_sum<CN>(a, l));
        pair u2[CN];
#pragma unroll
        for (int c = 0; c < CN; ++c) {
          const float x = __shfl_sync(0xffffffffu, u, c * (16 / CN), 16);
          u2[c] = pk(x, x);
        }
#pragma unroll
        for (int j = 0; j < J; ++j) {
          const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(kr + 64 * j);
          const ulonglong2 g = *reinterpret_cast<const ulonglong2*>(kr + S::kVec + 64 * j);
#pragma unroll
          for (int c = 0; c < CN; ++c) {
            s[c][j][0] = fma2(k.x, u2[c], mul2(g.x, s[c][j][0]));
            s[c][j][1] = fma2(k.y, u2[c], mul2(g.y, s[c][j][1]));
          }
        }
        o = fmaf(kq, u, scatter_sum<CN>(w, l));
      } else {
        pair w2[CN], v2[CN];
#pragma unroll
        for (int c = 0; c < CN; c += 4) {
          const float4 v = *reinterpret_cast<const float4*>(vt + i * S::kCols + col + c);
          v2[c] = pk(v.x, v.x); v2[c + 1] = pk(v.y, v.y); v2[c + 2] = pk(v.z, v.z); v2[c + 3] = pk(v.w, v.w);
        }
#pragma unroll
        for (int c = 0; c < CN; ++c) w2[c] = 0ull;
#pragma unroll
        for (int j = 0; j < J; ++j) {
          const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(kr + 64 * j);
          const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(kr + S::kVec + 64 * j);
#pragma unroll
          for (int c = 0; c < CN; ++c) {
            s[c][j][0] = fma2(k.x, v2[c], mul2(dec2, s[c][j][0]));
            s[c][j][1] = fma2(k.y, v2[c], mul2(dec2, s[c][j][1]));
            w2[c] = fma2(s[c][j][1], q.y, fma2(s[c][j][0], q.x, w2[c]));
          }
        }
        float w[CN];
#pragma unroll
        for (int c = 0; c < CN; ++c) w[c] = pair_sum(w2[c]);
        o = scatter_sum<CN>(w, l);
      }
      if (store_out) out0[static_cast<size_t>(t0 + i) * out_step] = o;
    }
    if (more) stage(smem + (cur ^ 1) * S::kStage);
    __syncthreads();
  }
  if (has) {
#pragma unroll
    for (int c = 0; c < CN; ++c) {
#pragma unroll
      for (int j = 0; j < J; ++j) {
        if (c0 + col + c < p.vdim && 4 * l + 64 * j < p.dimP) {
          ulonglong2 v;
          v.x = s[c][j][0];
          v.y = s[c][j][1];
          *reinterpret_cast<ulonglong2*>(st0 + c * p.dimP + 64 * j) = v;
        }
      }
    }
  }
}

// one token per sequence.  grid (ceil(vdim / (16 CN)), H, B), 128 threads: CN columns per thread
template <typename T, bool DELTA, int J, int CN>
__global__ void __launch_bounds__(kThreads)
step_kernel(ScanArgs p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int b = blockIdx.z, h = blockIdx.y;
  const int t = p.cu[b];
  if (p.cu[b + 1] <= t) return;
  const int slot = p.state_slots[b];
  const bool has = slot >= 0 && slot < p.num_slots;
  const bool load = has && p.kv_lens[b] > 1;
  __shared__ __align__(16) float kq_s[DELTA ? 4 : 2 * 32 * J];
  const int lane = threadIdx.x & 31, l = lane & 7;
  const int col = (blockIdx.x * 16 + (threadIdx.x >> 3)) * CN;
  const int hg = h / (p.H / p.G);
  float* st = p.state + ((static_cast<size_t>(has ? slot : 0) * p.H + h) * p.vdim + col) * p.dimP + 4 * l;
  float4 s[CN][J];
#pragma unroll
  for (int c = 0; c < CN; ++c)
#pragma unroll
    for (int j = 0; j < J; ++j)
      s[c][j] = load && col + c < p.vdim ? *reinterpret_cast<const float4*>(st + c * p.dimP + 32 * j)
                                         : make_float4(0.f, 0.f, 0.f, 0.f);
  float4 k[J], q[J];
  float v[CN], o[CN];
  if (DELTA) {
    const float* kp = p.k + (static_cast<size_t>(t) * p.G + hg) * p.dimP + 4 * l;
    const float* qp = p.q + (static_cast<size_t>(t) * p.G + hg) * p.dimP + 4 * l;
    const float* gp = p.g + (static_cast<size_t>(t) * p.H + h) * p.dimP + 4 * l;
    const float beta = p.beta[static_cast<size_t>(t) * p.H + h], kq = p.qk[static_cast<size_t>(t) * p.G + hg];
    float a[CN];
#pragma unroll
    for (int c = 0; c < CN; ++c) {
      v[c] = col + c < p.vdim ? p.v[(static_cast<size_t>(t) * p.H + h) * p.vdim + col + c] : 0.f;
      a[c] = o[c] = 0.f;
    }
#pragma unroll
    for (int j = 0; j < J; ++j) {
      k[j] = *reinterpret_cast<const float4*>(kp + 32 * j);
      q[j] = *reinterpret_cast<const float4*>(qp + 32 * j);
      const float4 g = *reinterpret_cast<const float4*>(gp + 32 * j);
#pragma unroll
      for (int c = 0; c < CN; ++c) {
        const float4 x = s[c][j] = mul4(g, s[c][j]);
        a[c] = fmaf(x.x, k[j].x, fmaf(x.y, k[j].y, fmaf(x.z, k[j].z, fmaf(x.w, k[j].w, a[c]))));
        o[c] = fmaf(x.x, q[j].x, fmaf(x.y, q[j].y, fmaf(x.z, q[j].z, fmaf(x.w, q[j].w, o[c]))));
      }
    }
#pragma unroll
    for (int c = 0; c < CN; ++c) {
      v[c] = beta * (v[c] - sum8(a[c]));                        // u
      o[c] = fmaf(kq, v[c], sum8(o[c]));
    }
#pragma unroll
    for (int c = 0; c < CN; ++c)
#pragma unroll
      for (int j = 0; j < J; ++j) {
        s[c][j].x = fmaf(k[j].x, v[c], s[c][j].x);
        s[c][j].y = fmaf(k[j].y, v[c], s[c][j].y);
        s[c][j].z = fmaf(k[j].z, v[c], s[c][j].z);
        s[c][j].w = fmaf(k[j].w, v[c], s[c][j].w);
      }
  } else {
    const T* row = static_cast<const T*>(p.proj) + static_cast<size_t>(t) * p.ld;
    const float dec = p.decay[h];
    // SiLU of the head's k and q once per block (the state is on its way meanwhile)
    for (int i = threadIdx.x; i < 16 * J; i += kThreads) {
      const int c4 = (i % (8 * J)) * 4;
      *reinterpret_cast<float4*>(kq_s + i * 4) = load4_silu(row + (i < 8 * J ? p.off_k : p.off_q) + h * p.dim, c4, p.dim, p.vec);
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < CN; ++c) {
      v[c] = col + c < p.vdim ? silu_f(to_f(row[p.off_v + h * p.vdim + col + c])) : 0.f;
      o[c] = 0.f;
    }
#pragma unroll
    for (int j = 0; j < J; ++j) {
      k[j] = *reinterpret_cast<const float4*>(kq_s + 4 * l + 32 * j);
      q[j] = *reinterpret_cast<const float4*>(kq_s + 32 * J + 4 * l + 32 * j);
#pragma unroll
      for (int c = 0; c < CN; ++c) {
        float4& x = s[c][j];
        x.x = fmaf(k[j].x, v[c], dec * x.x); o[c] = fmaf(x.x, q[j].x, o[c]);
        x.y = fmaf(k[j].y, v[c], dec * x.y); o[c] = fmaf(x.y, q[j].y, o[c]);
        x.z = fmaf(k[j].z, v[c], dec * x.z); o[c] = fmaf(x.z, q[j].z, o[c]);
        x.w = fmaf(k[j].w, v[c], dec * x.w); o[c] = fmaf(x.w, q[j].w, o[c]);
      }
    }
#pragma unroll
    for (int c = 0; c < CN; ++c) o[c] = sum8(o[c]);
  }
  float* out = p.out + (static_cast<size_t>(t) * p.H + h) * p.vdim + col;
#pragma unroll
  for (int c = 0; c < CN; ++c) {
    if (col + c >= p.vdim) continue;
    if (l == 0) out[c] = o[c];
    if (has) {
#pragma unroll
      for (int j = 0; j < J; ++j) *reinterpret_cast<float4*>(st + c * p.dimP + 32 * j) = s[c][j];
    }
  }
}

template <typename T, bool DELTA, int J, int CN>
int launch_scan(const ScanArgs& p, int B, cudaStream_t stream) {
  using S = ScanSmem<DELTA, J, CN>;
  auto kern = scan_kernel<T, DELTA, J, CN>;
  if (S::kBytes > 48 * 1024 &&
      cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, S::kBytes) != cudaSuccess)
    return -2;
  tgi::launch(kern, dim3((p.vdim + S::kCols - 1) / S::kCols, p.H, B), dim3(kThreads), S::kBytes, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T, bool DELTA, int J>
int run(const ScanArgs& p, int B, int max_q, cudaStream_t stream) {
  if (max_q == 1) {
    constexpr int CN = J <= 4 ? 4 : 2;
    tgi::launch(step_kernel<T, DELTA, J, CN>, dim3((p.vdim + 16 * CN - 1) / (16 * CN), p.H, B), dim3(kThreads), 0, stream, p);
  } else {
    // eight columns per sixteen lanes use shared memory best; four keep more schedulers busy when there are few columns
    constexpr int JS = (J + 1) / 2;
    const long long wide = static_cast<long long>(B) * p.H * ((p.vdim + 63) / 64);
    if constexpr (JS <= 2) {
      if (wide >= 200) return launch_scan<T, DELTA, JS, 8>(p, B, stream);
    }
    return launch_scan<T, DELTA, JS, 4>(p, B, stream);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T, bool DELTA>
int dispatch(const ScanArgs& p, int B, int max_q, cudaStream_t stream) {
  if (B <= 0 || max_q <= 0) return 0;
  if (B > 65535 || p.H > 65535 || p.H % p.G != 0 || p.dimP % 32 != 0 || p.dimP < p.dim) return -10;
  switch (p.dimP / 32) {
    case 1: return run<T, DELTA, 1>(p, B, max_q, stream);
    case 2: return run<T, DELTA, 2>(p, B, max_q, stream);
    case 3: return run<T, DELTA, 3>(p, B, max_q, stream);
    case 4: return run<T, DELTA, 4>(p, B, max_q, stream);
    case 5: case 6: return p.dimP == 192 ? run<T, DELTA, 6>(p, B, max_q, stream) : -12;
    case 8: return run<T, DELTA, 8>(p, B, max_q, stream);
    default: return -12;
  }
}

}  // namespace

extern "C" {

// Row pitch of a head's state and of its q / k / g vectors: the kernels exist for these widths.  0: too wide.
int tgi_recurrent_pitch(int dim) {
  for (int w : {32, 64, 96, 128, 192, 256})
    if (dim <= w) return w;
  return 0;
}

int tgi_delta_scan(const float* q, const float* k, const float* g, const float* v, const float* beta, const float* qk,
                   const int* cu, const int* kv_lens, const int* state_slots, float* state, float* out, int B, int max_q,
                   int num_slots, int G, int H, int dim, int dimP, int vdim, cudaStream_t stream) {
  ScanArgs p{};
  p.q = q; p.k = k; p.g = g; p.v = v; p.beta = beta; p.qk = qk;
  p.cu = cu; p.kv_lens = kv_lens; p.state_slots = state_slots;
  p.state = state; p.out = out;
  p.num_slots = num_slots; p.G = G; p.H = H; p.dim = dim; p.dimP = dimP; p.vdim = vdim;
  return dispatch<float, true>(p, B, max_q, stream);
}

int tgi_decay_scan(int f32, const void* proj, long long ld, int off_q, int off_k, int off_v, const float* decay, const int* cu,
                   const int* kv_lens, const int* state_slots, float* state, float* out, int B, int max_q, int num_slots,
                   int H, int dim, int dimP, int vdim, cudaStream_t stream) {
  ScanArgs p{};
  p.proj = proj; p.ld = ld; p.off_q = off_q; p.off_k = off_k; p.off_v = off_v; p.decay = decay;
  p.cu = cu; p.kv_lens = kv_lens; p.state_slots = state_slots;
  p.state = state; p.out = out;
  p.num_slots = num_slots; p.G = H; p.H = H; p.dim = dim; p.dimP = dimP; p.vdim = vdim;
  p.vec = dim % 4 == 0 && ld % 4 == 0 && off_q % 4 == 0 && off_k % 4 == 0 &&
          reinterpret_cast<uintptr_t>(proj) % (f32 ? 16 : 8) == 0;
  return f32 ? dispatch<float, false>(p, B, max_q, stream) : dispatch<bf16, false>(p, B, max_q, stream);
}

}  // extern "C"
