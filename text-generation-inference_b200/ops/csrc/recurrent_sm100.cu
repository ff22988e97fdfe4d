// Recurrent token mixers with a matrix state per head, S[dim x vdim] in fp32:
//
//   gated delta rule, one decay per key channel      S <- g * S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   the same with one decay per head                 (g a scalar)
//   linear attention with a fixed decay per head     S <- d S + k v^T;                                    o = S^T q
//                                                    (q, k, v as projected or after SiLU, k times a factor)
//
// The columns of S never meet: column j of a head needs k, q, g of the head and only v_j of its own.
//
// scan_kernel walks the tokens a sequence brings in this step with the state in registers (one load and one store of
// the state per step, whatever the number of tokens), four tokens at a time.  With G_i the product of the decays since
// the start of a block (elementwise over key channels), S the state before it and D_ji the decays after token j up to i:
//   u_i = beta_i (v_i - S^T (G_i k_i) - sum_{j<i} (k_j . D_ji k_i) u_j)
//   o_i = S^T (G_i q_i) + sum_{j<=i} (k_j . D_ji q_i) u_j
//   S  <- G_3 S + sum_j (D_j3 k_j) u_j^T
// which is the token-by-token rule with all products on the old state: they are independent, one reduction latency is
// paid per block, and the scalars are shared by all columns.  Only products of decays appear, never quotients, so a
// channel that forgets within a token loses nothing.  (One decay per head: G and D are scalars, taken out of the products,
// so that k and q are staged as they are.  Fixed decay: u = v, D and G are powers of d.)
// L lanes share CN columns, lane l holding rows 4 (l + L j) + (0..3) of each: a 16-byte shared-memory read feeds 4 CN
// multiply-adds, done in pairs (fma.rn.f32x2).  The sums of the CN columns are reduced by halving exchanges, after which
// every lane owns one column.  The vectors and scalars of the next tile of kTile tokens are prepared from registers
// while the current one runs.
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
// fixed decay (of SiLU'd vectors, of vectors as projected), delta rule with a decay per channel, per head
enum { kFixed = 0, kChannel = 1, kHead = 2, kPlain = 3 };
__host__ __device__ constexpr bool is_delta(int mode) { return mode == kChannel || mode == kHead; }
constexpr int kThreads = 128;

__device__ __forceinline__ float to_f(float x) { return x; }
__device__ __forceinline__ float to_f(bf16 x) { return __bfloat162float(x); }
// bf16 inputs: the hardware exponential and reciprocal (a few ulp of fp32)
template <typename T>
__device__ __forceinline__ float silu_t(float x) { return x / (1.f + expf(-x)); }
template <>
__device__ __forceinline__ float silu_t<bf16>(float x) { return __fdividef(x, 1.f + __expf(-x)); }

struct ScanArgs {
  // delta rule: fp32 q, k [T, G, dimP], g [T, H, dimP] (one decay per head: [T, H]), v [T, H, vdim], beta [T, H], qk = q . k [T, G]
  const float *q, *k, *g, *v, *beta, *qk;
  // linear attention: proj [T, ld] with q, k (H x dim) and v (H x vdim) at off_q, off_k, off_v (SiLU, if any, applied here)
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
  float k_scale;                  // linear attention: factor of k
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

// A second read of shared memory that the compiler must not replace by keeping the first one in registers
__device__ __forceinline__ ulonglong2 reread(const float* p) {
  ulonglong2 v;
  asm volatile("ld.volatile.shared.v2.u64 {%0, %1}, [%2];"
               : "=l"(v.x), "=l"(v.y)
               : "r"(static_cast<uint32_t>(__cvta_generic_to_shared(p))));
  return v;
}

// Sums of CN values over L lanes; lane l ends with the total of value l / (L / CN).
template <int CN, int L>
__device__ __forceinline__ float scatter_sum(float (&v)[CN], int l) {
  int m = L / 2;
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
// Two neighbouring elements as they are loaded, kept in the registers of a float2 until they are converted.
template <typename T>
struct PairOf;
template <>
struct PairOf<float> {
  using type = float2;
  static __device__ __forceinline__ float2 hold(float2 v) { return v; }
  static __device__ __forceinline__ float2 value(float2 v) { return v; }
};
template <>
struct PairOf<bf16> {
  using type = uint32_t;
  static __device__ __forceinline__ float2 hold(uint32_t v) { return make_float2(__uint_as_float(v), 0.f); }
  static __device__ __forceinline__ float2 value(float2 v) {
    const uint32_t w = __float_as_uint(v.x);
    return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w));
  }
};
template <typename T, int MODE>
__device__ __forceinline__ float act_t(float x) { return MODE == kFixed ? silu_t<T>(x) : x; }
// columns c .. c + 3 of a head after SiLU (if any) times f, zero past `dim`; `vec`: the four may be read at once
template <typename T, int MODE>
__device__ __forceinline__ float4 load4_act(const T* p, int c, int dim, bool vec, float f) {
  if (vec && c < dim) {
    const float4 x = raw4(p + c);
    return make_float4(f * act_t<T, MODE>(x.x), f * act_t<T, MODE>(x.y), f * act_t<T, MODE>(x.z), f * act_t<T, MODE>(x.w));
  }
  float v[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) v[i] = c + i < dim ? f * act_t<T, MODE>(to_f(p[c + i])) : 0.f;
  return make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }

constexpr int kBlock = 4;         // tokens whose products with the state are formed together

// (first, last) token of the 16 scalars of a block, a nibble each: ten with queries, six with keys
constexpr unsigned long long kPairFirst = 0x2110003221110000ull, kPairLast = 0x3323213323213210ull;

// L lanes share CN columns of a head whose vectors are 64 J wide
template <int MODE, int J, int L, int CN>
struct ScanCfg {
  static constexpr int kRow = 64 * J;
  static constexpr int kQuads = 16 * J / L;                     // 16-byte pieces of a column per lane
  static constexpr int kCols = kThreads / L * CN;               // columns of a CTA
  static constexpr bool kWide = MODE == kChannel;
  static constexpr int kRows = kWide ? 13 : 8;                  // vectors of a block: q', k^ (x 4 each) | + k' (x 4), decay
  static constexpr int kQ = 0, kEnd = 4, kK = kWide ? 8 : 4, kG = kWide ? 12 : 0;      // first row of each kind
  static constexpr int kVecs = 2 * kRows * kRow;                // floats: two blocks per tile
  static constexpr int kOffV = kVecs, kOffBeta = kOffV + kTile * kCols, kOffGate = kOffBeta + kTile,
                       kOffScal = kOffGate + kTile, kOffPart = kOffScal + 32, kStage = kOffPart + 2 * J * 16;
  static constexpr int kBytes = 2 * kStage * 4;
};

// grid (ceil(vdim / kCols), H, B), 128 threads.  VEC: the heads of proj may be read in aligned pairs.
template <typename T, int MODE, bool VEC, int J, int L, int CN>
__global__ void __launch_bounds__(kThreads)
scan_kernel(ScanArgs p) {
  constexpr bool DELTA = is_delta(MODE), WIDE = MODE == kChannel, HEAD = MODE == kHead;
  tgi::pdl_wait();
  tgi::pdl_trigger();
  extern __shared__ __align__(16) float smem[];
  using S = ScanCfg<MODE, J, L, CN>;
  constexpr int kItems = 64 * J;                                // (block, channel pair) items of a tile
  constexpr int NI = (kItems + kThreads - 1) / kThreads;
  constexpr int NV = kTile * S::kCols / kThreads;
  constexpr int NQ = S::kQuads;
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * S::kCols;
  const int begin = p.cu[b], n = p.cu[b + 1] - begin;
  if (n <= 0) return;
  const int start = p.kv_lens[b] - n, slot = p.state_slots[b];
  const bool has = slot >= 0 && slot < p.num_slots;
  const int tid = threadIdx.x, l = tid % L;
  const int col = (tid / L) * CN;                               // first column of this group, inside the tile
  const int mine = l / (L / CN);                                // the column whose sums this lane ends up with
  const int hg = h / (p.H / p.G);
  float* st0 = p.state + ((static_cast<size_t>(has ? slot : 0) * p.H + h) * p.vdim + c0 + col) * p.dimP + 4 * l;
  const bool store_out = l % (L / CN) == 0 && c0 + col + mine < p.vdim;
  const float dec = DELTA ? 1.f : p.decay[h];

  pair s[CN][NQ][2];
#pragma unroll
  for (int c = 0; c < CN; ++c) {
#pragma unroll
    for (int j = 0; j < NQ; ++j) {
      s[c][j][0] = s[c][j][1] = 0ull;
      if (has && start > 0 && c0 + col + c < p.vdim && 4 * (l + L * j) < p.dimP) {
        const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(st0 + c * p.dimP + 4 * L * j);
        s[c][j][0] = v.x;
        s[c][j][1] = v.y;
      }
    }
  }

  // two channels of the four tokens of a block, as they come from memory; pointers advance by a tile
  using E2 = typename PairOf<T>::type;
  float2 rk[NI][kBlock], rq[NI][kBlock], rg[WIDE ? NI : 1][kBlock];
  T rv[DELTA ? 1 : NV];
  float rvf[DELTA ? NV : 1], rb = 0.f, rh = 1.f;
  const size_t sk = DELTA ? static_cast<size_t>(p.G) * p.dimP : static_cast<size_t>(p.ld);   // token pitch of q and k
  const size_t sg = static_cast<size_t>(p.H) * p.dimP, sv = static_cast<size_t>(p.H) * p.vdim;
  const T* const proj = static_cast<const T*>(p.proj);
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int it = tid + i * kThreads, tb = t0 + it / (32 * J) * kBlock, c2 = (it % (32 * J)) * 2;
      const bool in = it < kItems && c2 < (DELTA ? p.dimP : p.dim);
      const size_t tok = begin + tb;
      const float* fk = p.k + tok * sk + hg * p.dimP + c2;
      const float* fq = p.q + tok * sk + hg * p.dimP + c2;
      const float* fg = p.g + tok * sg + h * p.dimP + c2;
      const T* xk = proj + tok * sk + p.off_k + h * p.dim + c2;
      const T* xq = proj + tok * sk + p.off_q + h * p.dim + c2;
#pragma unroll
      for (int e = 0; e < kBlock; ++e) {
        const bool ok = in && tb + e < n;
        if (DELTA) {
          rk[i][e] = rq[i][e] = make_float2(0.f, 0.f);
          if (WIDE) rg[WIDE ? i : 0][e] = make_float2(1.f, 1.f);
          if (ok) {
            rk[i][e] = *reinterpret_cast<const float2*>(fk + e * sk);
            rq[i][e] = *reinterpret_cast<const float2*>(fq + e * sk);
            if (WIDE) rg[WIDE ? i : 0][e] = *reinterpret_cast<const float2*>(fg + e * sg);
          }
        } else if (VEC) {
          E2 a = E2(), c = E2();
          if (ok) {
            a = *reinterpret_cast<const E2*>(xk + e * sk);
            c = *reinterpret_cast<const E2*>(xq + e * sk);
          }
          // kept as loaded: the conversion waits for the data, and belongs to `stage`
          rk[i][e] = PairOf<T>::hold(a);
          rq[i][e] = PairOf<T>::hold(c);
        } else {
          const bool two = c2 + 1 < p.dim;
          rk[i][e] = make_float2(ok ? to_f(xk[e * sk]) : 0.f, ok && two ? to_f(xk[e * sk + 1]) : 0.f);
          rq[i][e] = make_float2(ok ? to_f(xq[e * sk]) : 0.f, ok && two ? to_f(xq[e * sk + 1]) : 0.f);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int it = tid + i * kThreads, tk = t0 + it / S::kCols, c = c0 + it % S::kCols;
      const bool ok = tk < n && c < p.vdim;
      const size_t tok = begin + tk;
      if (DELTA) {
        rvf[DELTA ? i : 0] = 0.f;
        if (ok) rvf[DELTA ? i : 0] = p.v[tok * sv + h * p.vdim + c];
      } else {
        rv[DELTA ? 0 : i] = T(0.f);
        if (ok) rv[DELTA ? 0 : i] = proj[tok * p.ld + p.off_v + h * p.vdim + c];
      }
    }
    if (DELTA && tid < kTile) rb = t0 + tid < n ? p.beta[static_cast<size_t>(begin + t0 + tid) * p.H + h] : 0.f;
    if (HEAD && tid < kTile) rh = t0 + tid < n ? p.g[static_cast<size_t>(begin + t0 + tid) * p.H + h] : 1.f;
  };
  // vectors and partial scalar products of the fetched tile (tokens t0 ..) -> shared memory
  auto stage = [&](float* d, int t0) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int it = tid + i * kThreads, blk = it / (32 * J), c2 = (it % (32 * J)) * 2;
      if (it >= kItems) continue;                               // warp-uniform
      float2 k[kBlock], q[kBlock], g[kBlock];
      const int cnt = min(kBlock, n - t0 - blk * kBlock);       // <= 0: a block past the end, nothing reads it
#pragma unroll
      for (int e = 0; e < kBlock; ++e) {
        k[e] = rk[i][e];
        q[e] = rq[i][e];
        if (WIDE) {
          g[e] = rg[WIDE ? i : 0][e];
        } else if (HEAD) {
          g[e] = make_float2(1.f, 1.f);                         // decays are applied to the sums
        } else {
          if (VEC) {
            k[e] = PairOf<T>::value(k[e]);
            q[e] = PairOf<T>::value(q[e]);
          }
          k[e] = make_float2(act_t<T, MODE>(k[e].x), act_t<T, MODE>(k[e].y));    // SiLU(0) = 0: absent tokens and channels stay 0
          q[e] = make_float2(act_t<T, MODE>(q[e].x), act_t<T, MODE>(q[e].y));
          if (MODE == kPlain) k[e] = make_float2(p.k_scale * k[e].x, p.k_scale * k[e].y);
          g[e].x = g[e].y = e < cnt ? dec : 1.f;
        }
      }
      float* r = d + blk * S::kRows * S::kRow + c2;
      auto row = [&](int x, float2 v) { *reinterpret_cast<float2*>(r + x * S::kRow) = v; };
      auto mul = [](float2 a, float2 b) { return make_float2(a.x * b.x, a.y * b.y); };
      auto dot = [](float2 a, float2 b) { return a.x * b.x + a.y * b.y; };
      // decays since the start of the block, and from a token to its end
      float2 to[kBlock], from[kBlock];
      to[0] = g[0];
#pragma unroll
      for (int e = 1; e < kBlock; ++e) to[e] = mul(to[e - 1], g[e]);
      from[kBlock - 1] = make_float2(1.f, 1.f);
#pragma unroll
      for (int e = kBlock - 2; e >= 0; --e) from[e] = mul(from[e + 1], g[e + 1]);
#pragma unroll
      for (int e = 0; e < kBlock; ++e) {
        row(S::kQ + e, mul(to[e], q[e]));
        row(S::kEnd + e, mul(from[e], k[e]));
        if (WIDE) row(S::kK + e, mul(to[e], k[e]));
      }
      if (WIDE) row(S::kG, to[kBlock - 1]);
      // token a's key, decayed to token e, times e's query (10 sums over channels) and e's key (6 sums)
      float sc[16];
      int at = 0;
#pragma unroll
      for (int a = 0; a < kBlock; ++a) {
        float2 kd = k[a];
        sc[at++] = dot(kd, q[a]);
#pragma unroll
        for (int e = a + 1; e < kBlock; ++e) {
          kd = mul(kd, g[e]);
          sc[at++] = dot(kd, q[e]);
          sc[10 + a * (7 - a) / 2 + (e - a - 1)] = DELTA ? dot(kd, k[e]) : 0.f;
        }
      }
      // over the warp: lanes 2 x and 2 x + 1 end with sum x
#pragma unroll
      for (int half = 8, m = 16; half >= 1; half /= 2, m >>= 1) {
        const bool up = tid & m;
#pragma unroll
        for (int a = 0; a < half; ++a) {
          const float give = up ? sc[a] : sc[a + half], keep = up ? sc[a + half] : sc[a];
          sc[a] = keep + __shfl_xor_sync(0xffffffffu, give, m);
        }
      }
      sc[0] += __shfl_xor_sync(0xffffffffu, sc[0], 1);
      if ((tid & 1) == 0) d[S::kOffPart + (blk * J + c2 / 64) * 16 + (tid & 31) / 2] = sc[0];
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
      d[S::kOffV + tid + i * kThreads] = DELTA ? rvf[DELTA ? i : 0] : act_t<T, MODE>(to_f(rv[DELTA ? 0 : i]));
    if (DELTA && tid < kTile) d[S::kOffBeta + tid] = rb;
    if (HEAD && tid < kTile) d[S::kOffGate + tid] = rh;
  };
  // the sums of the warps that shared a block
  auto finish = [&](float* d) {
    if (tid < 32) {
      float x = 0.f;
#pragma unroll
      for (int j = 0; j < J; ++j) x += d[S::kOffPart + ((tid >> 4) * J + j) * 16 + (tid & 15)];
      if (HEAD) {                                               // decay after the first token of the pair up to the last
        const int first = kPairFirst >> (4 * (tid & 15)) & 15, last = kPairLast >> (4 * (tid & 15)) & 15;
#pragma unroll
        for (int e = 1; e < kBlock; ++e)
          if (e > first && e <= last) x *= d[S::kOffGate + (tid >> 4) * kBlock + e];
      }
      d[S::kOffScal + tid] = x;
    }
  };
  fetch(0);
  stage(smem, 0);
  __syncthreads();
  finish(smem);
  __syncthreads();
  float* const out0 = p.out + (static_cast<size_t>(begin) * p.H + h) * p.vdim + c0 + col + mine;
  for (int t0 = 0, cur = 0; t0 < n; t0 += kTile, cur ^= 1) {
    const bool more = t0 + kTile < n;
    if (more) fetch(t0 + kTile);
    const float* d = smem + cur * S::kStage;
#pragma unroll 1
    for (int blk = 0; blk < 2 && t0 + blk * kBlock < n; ++blk) {
      const float* r = d + blk * S::kRows * S::kRow + 4 * l;
      const float* vt = d + S::kOffV + blk * kBlock * S::kCols + col;
      float w[kBlock], u[kBlock], since[kBlock];                // decay of the head since the start of the block
      float4 gate = make_float4(1.f, 1.f, 1.f, 1.f);
      if (HEAD) {
        gate = *reinterpret_cast<const float4*>(d + S::kOffGate + blk * kBlock);
        since[0] = gate.x;
        since[1] = since[0] * gate.y;
        since[2] = since[1] * gate.z;
        since[3] = since[2] * gate.w;
      }
      // products of every token of the block with the state before it
#pragma unroll
      for (int e = 0; e < kBlock; ++e) {
        float a[CN];
        pair x2[CN];
        u[e] = vt[e * S::kCols + mine];
        if (DELTA) {
#pragma unroll
          for (int j = 0; j < NQ; ++j) {
            const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(r + (S::kK + e) * S::kRow + 4 * L * j);
#pragma unroll
            for (int c = 0; c < CN; ++c)
              x2[c] = fma2(s[c][j][1], k.y, j == 0 ? mul2(s[c][j][0], k.x) : fma2(s[c][j][0], k.x, x2[c]));
          }
#pragma unroll
          for (int c = 0; c < CN; ++c) a[c] = pair_sum(x2[c]);
          const float r0 = scatter_sum<CN, L>(a, l);
          u[e] = HEAD ? fmaf(-since[e], r0, u[e]) : u[e] - r0;
        }
#pragma unroll
        for (int j = 0; j < NQ; ++j) {
          const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(r + (S::kQ + e) * S::kRow + 4 * L * j);
#pragma unroll
          for (int c = 0; c < CN; ++c)
            x2[c] = fma2(s[c][j][1], q.y, j == 0 ? mul2(s[c][j][0], q.x) : fma2(s[c][j][0], q.x, x2[c]));
        }
#pragma unroll
        for (int c = 0; c < CN; ++c) a[c] = pair_sum(x2[c]);
        w[e] = scatter_sum<CN, L>(a, l);
        if (HEAD) w[e] *= since[e];
      }
      // what the tokens write, first to last, and what they read of each other
      const float4* sc = reinterpret_cast<const float4*>(d + S::kOffScal + blk * 16);
      const float4 s0 = sc[0], s1 = sc[1], s2 = sc[2];          // q: 00 01 02 03 | 11 12 13 22 | 23 33, k: 01 02
      if (DELTA) {
        const float4 s3 = sc[3];                                // k: 03 12 13 23
        const float4 beta = *reinterpret_cast<const float4*>(d + S::kOffBeta + blk * kBlock);
        u[0] *= beta.x;
        u[1] = beta.y * fmaf(-s2.z, u[0], u[1]);
        u[2] = beta.z * fmaf(-s3.y, u[1], fmaf(-s2.w, u[0], u[2]));
        u[3] = beta.w * fmaf(-s3.w, u[2], fmaf(-s3.z, u[1], fmaf(-s3.x, u[0], u[3])));
      }
      w[0] = fmaf(s0.x, u[0], w[0]);
      w[1] = fmaf(s0.y, u[0], fmaf(s1.x, u[1], w[1]));
      w[2] = fmaf(s0.z, u[0], fmaf(s1.y, u[1], fmaf(s1.w, u[2], w[2])));
      w[3] = fmaf(s0.w, u[0], fmaf(s1.z, u[1], fmaf(s2.x, u[2], fmaf(s2.y, u[3], w[3]))));
      // the state after the block
      const int cnt = min(kBlock, n - t0 - blk * kBlock);
      if (WIDE) {
#pragma unroll
        for (int j = 0; j < NQ; ++j) {
          const ulonglong2 g = *reinterpret_cast<const ulonglong2*>(r + S::kG * S::kRow + 4 * L * j);
#pragma unroll
          for (int c = 0; c < CN; ++c) {
            s[c][j][0] = mul2(g.x, s[c][j][0]);
            s[c][j][1] = mul2(g.y, s[c][j][1]);
          }
        }
      } else {
        const float d2 = dec * dec;
        const float f = HEAD ? since[3] : (cnt == 4 ? d2 * d2 : (cnt == 3 ? d2 * dec : (cnt == 2 ? d2 : dec)));
        const pair f2 = pk(f, f);
#pragma unroll
        for (int j = 0; j < NQ; ++j) {
#pragma unroll
          for (int c = 0; c < CN; ++c) {
            s[c][j][0] = mul2(f2, s[c][j][0]);
            s[c][j][1] = mul2(f2, s[c][j][1]);
          }
        }
      }
      if (HEAD) {                                               // what is left of each write at the end of the block
        u[2] *= gate.w;
        u[1] *= gate.z * gate.w;
        u[0] *= gate.y * gate.z * gate.w;
      }
#pragma unroll
      for (int e = 0; e < kBlock; ++e) {
        pair u2[CN];
#pragma unroll
        for (int c = 0; c < CN; ++c) {
          const float x = DELTA ? __shfl_sync(0xffffffffu, u[e], c * (L / CN), L) : vt[e * S::kCols + c];
          u2[c] = pk(x, x);
        }
#pragma unroll
        for (int j = 0; j < NQ; ++j) {
          const float* kp = r + (S::kEnd + e) * S::kRow + 4 * L * j;
          const ulonglong2 k = HEAD ? reread(kp) : *reinterpret_cast<const ulonglong2*>(kp);
#pragma unroll
          for (int c = 0; c < CN; ++c) {
            s[c][j][0] = fma2(k.x, u2[c], s[c][j][0]);
            s[c][j][1] = fma2(k.y, u2[c], s[c][j][1]);
          }
        }
      }
      if (store_out) {
        float* o = out0 + (t0 + blk * kBlock) * sv;
#pragma unroll
        for (int e = 0; e < kBlock; ++e)
          if (e < cnt) o[e * sv] = w[e];
      }
    }
    if (more) {
      stage(smem + (cur ^ 1) * S::kStage, t0 + kTile);
      __syncthreads();
      finish(smem + (cur ^ 1) * S::kStage);
    }
    __syncthreads();
  }
  if (has) {
#pragma unroll
    for (int c = 0; c < CN; ++c) {
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        if (c0 + col + c < p.vdim && 4 * (l + L * j) < p.dimP) {
          ulonglong2 v;
          v.x = s[c][j][0];
          v.y = s[c][j][1];
          *reinterpret_cast<ulonglong2*>(st0 + c * p.dimP + 4 * L * j) = v;
        }
      }
    }
  }
}

// one token per sequence.  grid (ceil(vdim / (16 CN)), H, B), 128 threads: CN columns per thread
template <typename T, int MODE, int J, int CN>
__global__ void __launch_bounds__(kThreads)
step_kernel(ScanArgs p) {
  constexpr bool DELTA = is_delta(MODE), HEAD = MODE == kHead;
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
    const float gh = HEAD ? p.g[static_cast<size_t>(t) * p.H + h] : 1.f;
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
      const float4 g = HEAD ? make_float4(gh, gh, gh, gh) : *reinterpret_cast<const float4*>(gp + 32 * j);
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
    // the head's k and q once per block (the state is on its way meanwhile)
    for (int i = threadIdx.x; i < 16 * J; i += kThreads) {
      const int c4 = (i % (8 * J)) * 4;
      *reinterpret_cast<float4*>(kq_s + i * 4) = load4_act<T, MODE>(row + (i < 8 * J ? p.off_k : p.off_q) + h * p.dim, c4, p.dim,
                                                                         p.vec, MODE == kPlain && i < 8 * J ? p.k_scale : 1.f);
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < CN; ++c) {
      v[c] = col + c < p.vdim ? act_t<T, MODE>(to_f(row[p.off_v + h * p.vdim + col + c])) : 0.f;
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

template <typename T, int MODE, bool VEC, int J, int L, int CN>
int launch_scan(const ScanArgs& p, int B, cudaStream_t stream) {
  using S = ScanCfg<MODE, J, L, CN>;
  auto kern = scan_kernel<T, MODE, VEC, J, L, CN>;
  if (S::kBytes > 48 * 1024 &&
      cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, S::kBytes) != cudaSuccess)
    return -2;
  tgi::launch(kern, dim3((p.vdim + S::kCols - 1) / S::kCols, p.H, B), dim3(kThreads), S::kBytes, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T, int MODE, int J>
int run(const ScanArgs& p, int B, int max_q, cudaStream_t stream) {
  constexpr bool DELTA = is_delta(MODE);
  if (max_q == 1) {
    constexpr int CN = J <= 4 ? 4 : 2;
    tgi::launch(step_kernel<T, MODE, J, CN>, dim3((p.vdim + 16 * CN - 1) / (16 * CN), p.H, B), dim3(kThreads), 0, stream, p);
  } else {
    // Wide lanes and few columns keep every scheduler busy when there are few sequences; many columns per lane need
    // fewer shared-memory reads and shuffles per column.  Measured, 32 heads of 128 x 128, delta rule, us (16 lanes x 4
    // columns, 16 x 8, 4 x 4): 1 sequence of 8192 tokens 1973, 2593, 3816; 2 x 4096 1399, 1300, 1913; 4 x 2048 1235,
    // 1045, 962; 16 x 512 1041, 845, 813.  Fixed decay: 2418, 3006, 4141; 1498, 1508, 2076; 1146, 990, 1043; 984, 771, 752.
    constexpr int JS = (J + 1) / 2;
    if (DELTA || p.vec) {
      if constexpr (JS <= 2) {
        const long long heads = static_cast<long long>(B) * p.H;
        if (heads * ((p.vdim + 127) / 128) >= (DELTA ? 128 : 192)) return launch_scan<T, MODE, true, JS, 4, 4>(p, B, stream);
        if (heads * ((p.vdim + 63) / 64) >= 128) return launch_scan<T, MODE, true, JS, 16, 8>(p, B, stream);
      }
      return launch_scan<T, MODE, true, JS, 16, 4>(p, B, stream);
    }
    if constexpr (!DELTA) return launch_scan<T, MODE, false, JS, 16, 4>(p, B, stream);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T, int MODE>
int dispatch(const ScanArgs& p, int B, int max_q, cudaStream_t stream) {
  if (B <= 0 || max_q <= 0) return 0;
  if (B > 65535 || p.H > 65535 || p.H % p.G != 0 || p.dimP % 32 != 0 || p.dimP < p.dim) return -10;
  switch (p.dimP / 32) {
    case 1: return run<T, MODE, 1>(p, B, max_q, stream);
    case 2: return run<T, MODE, 2>(p, B, max_q, stream);
    case 3: return run<T, MODE, 3>(p, B, max_q, stream);
    case 4: return run<T, MODE, 4>(p, B, max_q, stream);
    case 5: case 6: return p.dimP == 192 ? run<T, MODE, 6>(p, B, max_q, stream) : -12;
    case 8: return run<T, MODE, 8>(p, B, max_q, stream);
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

// `head_decay`: g is [T, H] instead of [T, H, dimP]
int tgi_delta_scan(const float* q, const float* k, const float* g, const float* v, const float* beta, const float* qk,
                   const int* cu, const int* kv_lens, const int* state_slots, float* state, float* out, int B, int max_q,
                   int num_slots, int G, int H, int dim, int dimP, int vdim, int head_decay, cudaStream_t stream) {
  ScanArgs p{};
  p.q = q; p.k = k; p.g = g; p.v = v; p.beta = beta; p.qk = qk;
  p.cu = cu; p.kv_lens = kv_lens; p.state_slots = state_slots;
  p.state = state; p.out = out;
  p.num_slots = num_slots; p.G = G; p.H = H; p.dim = dim; p.dimP = dimP; p.vdim = vdim;
  return head_decay ? dispatch<float, kHead>(p, B, max_q, stream) : dispatch<float, kChannel>(p, B, max_q, stream);
}

// `silu`: q, k and v go through SiLU (and k_scale is 1); otherwise k is multiplied by k_scale
int tgi_decay_scan(int f32, const void* proj, long long ld, int off_q, int off_k, int off_v, const float* decay, const int* cu,
                   const int* kv_lens, const int* state_slots, float* state, float* out, int B, int max_q, int num_slots,
                   int H, int dim, int dimP, int vdim, int silu, float k_scale, cudaStream_t stream) {
  ScanArgs p{};
  if (silu && k_scale != 1.f) return -13;                   // no instance
  p.k_scale = k_scale;
  p.proj = proj; p.ld = ld; p.off_q = off_q; p.off_k = off_k; p.off_v = off_v; p.decay = decay;
  p.cu = cu; p.kv_lens = kv_lens; p.state_slots = state_slots;
  p.state = state; p.out = out;
  p.num_slots = num_slots; p.G = H; p.H = H; p.dim = dim; p.dimP = dimP; p.vdim = vdim;
  p.vec = dim % 4 == 0 && ld % 4 == 0 && off_q % 4 == 0 && off_k % 4 == 0 &&
          reinterpret_cast<uintptr_t>(proj) % (f32 ? 16 : 8) == 0;
  if (silu) return f32 ? dispatch<float, kFixed>(p, B, max_q, stream) : dispatch<bf16, kFixed>(p, B, max_q, stream);
  return f32 ? dispatch<float, kPlain>(p, B, max_q, stream) : dispatch<bf16, kPlain>(p, B, max_q, stream);
}

}  // extern "C"
