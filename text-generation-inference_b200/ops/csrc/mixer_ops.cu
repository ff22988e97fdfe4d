// Kernels around the token mixers of hybrid decoders (attention layers between recurrent ones), each in a bf16 and
// an fp32 build of the activations:
//   residual add (fp32 stream) of one or two block outputs + one or two RMSNorms or a LayerNorm, optional row gather
//   embedding gather into the fp32 residual stream
//   element-wise activation of a non-gated feed-forward, act(gate) * up of a gated one
//   [causal short convolution ->] RoPE -> per-head RMS of q and k -> value mixing -> paged K / V store
//   paged attention for any head size and for fp32 pages (the tensor-core kernels serve bf16 at 64 / 128 / 256)
//   causal short convolution + SiLU, unit norms, decays and write strengths of a gated delta rule
//   per-group RMSNorm x weight x sigmoid(gate) or SiLU(gate) on the output of a recurrent mixer
//
// Norms, angles, scores, decays and the residual stream are fp32 in both builds; only matrix operands and what the
// matrix products return are bf16.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <type_traits>

#include "launch.cuh"
#include "mixer_util.cuh"

namespace {

using namespace mixer;

// ------------------------------------------------------------------------------------------------
// r = residual (fp32) + scale * (d1 + d2) -> RMSNorm(r) * (offset + w1) + b1 (`layer`: of r minus its mean), and the same with
// w2 and no bias.  One CTA per output row;
// `rows` (optional) picks the input row.  VPT float4 per thread stay in registers; VPT == 0: any width, read twice.
// ------------------------------------------------------------------------------------------------
template <typename T>
struct ResidualNorm {
  const T *d1, *d2;               // null: nothing to add
  const float* residual;
  const int* rows;
  const T *w1, *w2;               // w2 null: one norm
  const T* b1;                    // null: no bias
  T *o1, *o2;
  float* res_out;
  int H, layer;
  float eps, scale, offset;
};
template <typename T, int VPT>
__global__ void __launch_bounds__(1024)
residual_norm_kernel(ResidualNorm<T> p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  __shared__ float red[33];
  const int row = p.rows != nullptr ? p.rows[blockIdx.x] : blockIdx.x, H = p.H;
  const size_t in = static_cast<size_t>(row) * H, ob = static_cast<size_t>(blockIdx.x) * H;
  float sumsq = 0.f, sum = 0.f;
  if (VPT > 0) {
    float4 x[VPT > 0 ? VPT : 1];
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * 4;
      if (c < H) {
        float4 a = *reinterpret_cast<const float4*>(p.residual + in + c);
        if (p.d1 != nullptr) {
          float4 d = load4(p.d1 + in + c);
          if (p.d2 != nullptr) {
            const float4 e = load4(p.d2 + in + c);
            d.x += e.x; d.y += e.y; d.z += e.z; d.w += e.w;
          }
          a.x = fmaf(p.scale, d.x, a.x); a.y = fmaf(p.scale, d.y, a.y);
          a.z = fmaf(p.scale, d.z, a.z); a.w = fmaf(p.scale, d.w, a.w);
        }
        if (p.res_out != nullptr) store4(p.res_out + ob + c, a);
        x[i] = a;
        sumsq += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
        sum += (a.x + a.y) + (a.z + a.w);
      }
    }
    if (p.layer) {                                         // deviations, then their squares
      const float mean = block_sum(sum, red) / H;
      sumsq = 0.f;
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        if ((threadIdx.x + i * blockDim.x) * 4 < H) {
          x[i].x -= mean; x[i].y -= mean; x[i].z -= mean; x[i].w -= mean;
          sumsq += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
        }
      }
    }
    const float inv = 1.f / sqrtf(block_sum(sumsq, red) / H + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * 4;
      if (c < H) {
        const float4 y = make_float4(x[i].x * inv, x[i].y * inv, x[i].z * inv, x[i].w * inv);
        auto put_norm = [&](const T* weight, const T* bias, T* out) {
          const float4 w = load4(weight + c), b = bias != nullptr ? load4(bias + c) : make_float4(0.f, 0.f, 0.f, 0.f);
          store4(out + ob + c, make_float4(fmaf(y.x, p.offset + w.x, b.x), fmaf(y.y, p.offset + w.y, b.y),
                                           fmaf(y.z, p.offset + w.z, b.z), fmaf(y.w, p.offset + w.w, b.w)));
        };
        put_norm(p.w1, p.b1, p.o1);
        if (p.w2 != nullptr) put_norm(p.w2, nullptr, p.o2);
      }
    }
  } else {
    auto value = [&](int c) {
      float a = p.residual[in + c];
      if (p.d1 != nullptr) a = fmaf(p.scale, to_f(p.d1[in + c]) + (p.d2 != nullptr ? to_f(p.d2[in + c]) : 0.f), a);
      return a;
    };
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
      const float a = value(c);
      if (p.res_out != nullptr) p.res_out[ob + c] = a;
      sumsq += a * a;
      sum += a;
    }
    float mean = 0.f;
    if (p.layer) {
      mean = block_sum(sum, red) / H;
      sumsq = 0.f;
      for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float a = value(c) - mean;
        sumsq += a * a;
      }
    }
    const float inv = 1.f / sqrtf(block_sum(sumsq, red) / H + p.eps);
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
      const float y = (value(c) - mean) * inv;
      put(p.o1 + ob + c, fmaf(y, p.offset + to_f(p.w1[c]), p.b1 != nullptr ? to_f(p.b1[c]) : 0.f));
      if (p.w2 != nullptr) put(p.o2 + ob + c, y * (p.offset + to_f(p.w2[c])));
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
embed_residual_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out, int H, int vocab,
                      float scale) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int id = min(max(ids[blockIdx.x], 0), vocab - 1);
  const T* src = table + static_cast<size_t>(id) * H;
  float* dst = out + static_cast<size_t>(blockIdx.x) * H;
  if (H % 4 == 0) {
    for (int c = threadIdx.x * 4; c < H; c += blockDim.x * 4) {
      float4 v = load4(src + c);
      store4(dst + c, make_float4(v.x * scale, v.y * scale, v.z * scale, v.w * scale));
    }
  } else {
    for (int c = threadIdx.x; c < H; c += blockDim.x) dst[c] = to_f(src[c]) * scale;
  }
}

// ------------------------------------------------------------------------------------------------
// element-wise activation (codes as in the gated kernel: 0 silu, 1 gelu erf, 2 gelu tanh, 3 relu, 4 quick gelu,
// 5 squared relu), and act(gate) * up for fp32 and for widths the bf16 kernel does not take
// ------------------------------------------------------------------------------------------------
__device__ __forceinline__ float act_value(float x, int act) {
  switch (act) {
    case 0: return silu_f(x);
    case 1: return 0.5f * x * (1.f + erff(x * 0.70710678118654752f));
    case 2: return 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
    case 3: return fmaxf(x, 0.f);
    case 5: { const float y = fmaxf(x, 0.f); return y * y; }
    default: return x / (1.f + expf(-1.702f * x));
  }
}
template <typename T>
__global__ void __launch_bounds__(256)
act_mul_any_kernel(const T* __restrict__ in, T* __restrict__ out, long long n, int I, int act) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const long long stride = static_cast<long long>(gridDim.x) * blockDim.x;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n; i += stride) {
    const long long t = i / I, c = i - t * I;
    const T* row = in + t * 2 * I;
    put(out + i, act_value(to_f(row[c]), act) * to_f(row[I + c]));
  }
}
template <typename T>
__global__ void __launch_bounds__(256)
activation_kernel(const T* __restrict__ in, T* __restrict__ out, long long n, int act) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const long long stride = static_cast<long long>(gridDim.x) * blockDim.x;
  const long long first = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  const long long n4 = n / 4;
  for (long long i = first; i < n4; i += stride) {
    const float4 v = load4(in + i * 4);
    store4(out + i * 4, make_float4(act_value(v.x, act), act_value(v.y, act), act_value(v.z, act), act_value(v.w, act)));
  }
  for (long long i = n4 * 4 + first; i < n; i += stride) put(out + i, act_value(to_f(in[i]), act));
}

// ------------------------------------------------------------------------------------------------
// Short convolutions over time, one per channel, on three groups of columns of proj[T, ld] (q, k, v).  The previous
// taps - 1 inputs come from the step's rows or, before them, from the sequence's state [taps - 1][C] (C channels, q first,
// oldest input first); a sequence that starts at position 0 has zeros there.  In steps of single tokens the kernel that
// convolves also shifts the state (`update`), otherwise conv_state_kernel does it afterwards.
// ------------------------------------------------------------------------------------------------
struct ConvPast {
  const float* w;                 // [rows][C] taps, oldest first; null: no convolution
  const int *cu, *kv_lens, *slots;
  void* state;                    // [num_slots][taps - 1][C]
  int B, taps, C, num_slots, update;
};

// convolved value of channel `c` (column `col` of proj) for the token at row t, local index i of its sequence
template <typename T>
__device__ __forceinline__ float conv_value(const T* __restrict__ proj, long long ld, int col, int t, int i,
                                            const float* __restrict__ w, const T* __restrict__ st, int C, int c,
                                            int taps) {   // w: the channel's first tap, taps C floats apart
  float acc = 0.f;
  for (int j = 0; j < taps - 1; ++j) {             // tap j multiplies the input taps - 1 - j tokens back
    const int back = taps - 1 - j;
    float v = 0.f;
    if (i >= back) {
      v = to_f(proj[static_cast<size_t>(t - back) * ld + col]);
    } else if (st != nullptr) {
      v = to_f(st[static_cast<size_t>(taps - 1 + i - back) * C + c]);
    }
    acc = fmaf(w[static_cast<size_t>(j) * C], v, acc);
  }
  return fmaf(w[static_cast<size_t>(taps - 1) * C], to_f(proj[static_cast<size_t>(t) * ld + col]), acc);
}

// Weights and inputs of four neighbouring channels, TAPS <= 8; weights come as [TAPS][C] with absent taps zero.
template <typename T, int TAPS>
struct ShortConv {
  float4 w[TAPS];
  __device__ __forceinline__ void weights(const float* __restrict__ wt, int C, int c, bool ok) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
      w[j] = ok ? *reinterpret_cast<const float4*>(wt + static_cast<size_t>(j) * C + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  // inputs of the token at `row` (local index i of its sequence), oldest first: rows of this step, before them the
  // state (`st`, null: zeros)
  __device__ __forceinline__ void inputs(float4 (&x)[TAPS], const T* __restrict__ row, long long ld, int i,
                                         const T* __restrict__ st, int C, int taps, bool ok) const {
    const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i >= TAPS - 1) {               // warp-uniform
#pragma unroll
      for (int j = 0; j < TAPS; ++j) x[j] = ok ? load4(row - (TAPS - 1 - j) * ld) : z;
    } else {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const int back = TAPS - 1 - j;
        x[j] = z;
        if (!ok) continue;
        if (i >= back) x[j] = load4(row - back * ld);
        else if (st != nullptr && taps - 1 + i - back >= 0) x[j] = load4(st + static_cast<size_t>(taps - 1 + i - back) * C);
      }
    }
  }
  __device__ __forceinline__ float4 sum(const float4* x) const {         // x: TAPS inputs, oldest first
    float4 a = make_float4(w[0].x * x[0].x, w[0].y * x[0].y, w[0].z * x[0].z, w[0].w * x[0].w);
#pragma unroll
    for (int j = 1; j < TAPS; ++j) {
      a.x = fmaf(w[j].x, x[j].x, a.x);
      a.y = fmaf(w[j].y, x[j].y, a.y);
      a.z = fmaf(w[j].z, x[j].z, a.z);
      a.w = fmaf(w[j].w, x[j].w, a.w);
    }
    return a;
  }
  __device__ __forceinline__ float4 apply(const float4* x) const {       // followed by SiLU
    const float4 a = sum(x);
    return make_float4(silu_t<T>(a.x), silu_t<T>(a.y), silu_t<T>(a.z), silu_t<T>(a.w));
  }
  // the state after this token (single-token steps)
  static __device__ __forceinline__ void save(const float4 (&x)[TAPS], T* __restrict__ st, int C, int taps, bool ok) {
#pragma unroll
    for (int j = 1; j < TAPS; ++j) {
      const int e = j - 1 - (TAPS - taps);
      if (ok && e >= 0) store4(st + static_cast<size_t>(e) * C, x[j]);
    }
  }
};
__device__ __forceinline__ float dot4(float4 a, float4 b) { return a.x * b.x + a.y * b.y + a.z * b.z + a.w * b.w; }
__device__ __forceinline__ float decay_value(float z, float rate) {
  return expf(-rate * (z > 20.f ? z : log1pf(expf(z))));
}


// last taps - 1 inputs of every sequence that contributed tokens -> its convolution state.  Grid (channels / 256, B);
// channels 0 .. n0 - 1 are at column off0, the next n1 at off1, the rest at off2.
template <typename T>
__global__ void __launch_bounds__(256)
conv_state_kernel(const T* __restrict__ proj, long long ld, int n0, int n1, int off0, int off1, int off2, ConvPast p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int b = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int n = p.cu[b + 1] - p.cu[b], slot = p.slots[b];
  if (c >= p.C || n <= 0 || slot < 0 || slot >= p.num_slots) return;
  const int col = c < n0 ? off0 + c : (c < n0 + n1 ? off1 + c - n0 : off2 + c - n0 - n1);
  const bool fresh = p.kv_lens[b] - n <= 0;
  T* st = static_cast<T*>(p.state) + static_cast<size_t>(slot) * (p.taps - 1) * p.C + c;
  for (int j = 0; j < p.taps - 1; ++j) {            // ascending: entry j is only read by entries before it
    const int i = n - (p.taps - 1) + j;             // local index of the input that belongs at entry j
    T v = T(0.f);
    if (i >= 0) v = proj[static_cast<size_t>(p.cu[b] + i) * ld + col];
    else if (!fresh) v = st[static_cast<size_t>(p.taps - 1 + i) * p.C];
    st[static_cast<size_t>(j) * p.C] = v;
  }
}

// rows of the transposed convolution weights: absent taps in front are zero rows
int delta_tap_rows(int taps) { return taps <= 4 ? 4 : (taps <= 8 ? 8 : taps); }

// ------------------------------------------------------------------------------------------------
// Attention inputs.  proj[T, ld] holds q (Hq heads of `dim`), k (Hkv of `dim`) and v (Hkv of `vdim`) at columns
// 0, off_k, off_v.  One warp per (token, head): convolve over time (`conv`), rotate the first `rot` dimensions (pairs
// i, i + rot / 2, or 2i, 2i + 1 when `inter`), divide q and k by their root mean square over the head, mix v with the
// values of an earlier layer, and store k / v at the token's slot.  q_out rows are Dk wide; columns past `dim` are zeroed.
// The page pools are zero there already.
// ------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
attn_prep_kernel(const T* __restrict__ proj, long long ld, int off_k, int off_v, const int* __restrict__ positions,
                 const float* __restrict__ cos_sin, const int* __restrict__ slots, const T* __restrict__ v_first,
                 long long ld_first, float lambda, T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache,
                 int T_, int Hq, int Hkv, int dim, int vdim, int Dk, int Dv, int rot, int max_pos,
                 long long num_slots, int qk_norm, float eps, int inter, ConvPast cv) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int lane = threadIdx.x & 31;
  const int heads = Hq + 2 * Hkv;
  const long long job = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (job >= static_cast<long long>(T_) * heads) return;
  const int t = static_cast<int>(job / heads), h = static_cast<int>(job % heads);
  const long long slot = slots[t];
  const bool slot_ok = slot >= 0 && slot < num_slots;      // padding rows have slot -1
  const bool is_q = h < Hq, is_v = h >= Hq + Hkv;
  const int g = is_q ? h : (is_v ? h - Hq - Hkv : h - Hq), width = is_v ? vdim : dim;
  // first column and first channel of the head
  const int col = (is_q ? 0 : (is_v ? off_v : off_k)) + g * width;
  const int chan = is_v ? (Hq + Hkv) * dim + g * vdim : h * dim;
  const T* x = proj + static_cast<size_t>(t) * ld + col;
  T* st = nullptr;
  const T* old = nullptr;
  int local = 0;
  if (cv.w != nullptr) {
    const int b = sequence_of(cv.cu, cv.B, t), n = cv.cu[b + 1] - cv.cu[b], own = cv.slots[b];
    local = t - cv.cu[b];
    if (own >= 0 && own < cv.num_slots) st = static_cast<T*>(cv.state) + static_cast<size_t>(own) * (cv.taps - 1) * cv.C;
    old = cv.kv_lens[b] - n > 0 ? st : nullptr;
  }
  auto value = [&](int i) {
    return cv.w != nullptr ? conv_value(proj, ld, col + i, t, local, cv.w + chan + i, old, cv.C, chan + i, cv.taps) : to_f(x[i]);
  };
  auto shift_state = [&]() {                               // after every lane has read the state
    if (cv.w == nullptr || !cv.update || st == nullptr || cv.taps < 2) return;
    __syncwarp();
    for (int i = lane; i < width; i += 32) {
      for (int j = 0; j + 1 < cv.taps - 1; ++j)
        st[static_cast<size_t>(j) * cv.C + chan + i] = old != nullptr ? st[static_cast<size_t>(j + 1) * cv.C + chan + i] : T(0.f);
      st[static_cast<size_t>(cv.taps - 2) * cv.C + chan + i] = x[i];
    }
  };
  if (is_v) {
    if (slot_ok) {
      const T* f = v_first != nullptr ? v_first + static_cast<size_t>(t) * ld_first + static_cast<size_t>(g) * vdim : nullptr;
      for (int i = lane; i < vdim; i += 32) {
        float y = value(i);
        if (f != nullptr) y = (1.f - lambda) * y + lambda * to_f(f[i]);
        put(v_cache + (static_cast<size_t>(slot) * Hkv + g) * Dv + i, y);
      }
    }
    shift_state();
    return;
  }
  const int pos = min(max(positions[t], 0), max_pos - 1);
  const float* cs = cos_sin + static_cast<size_t>(pos) * rot;
  const int rh = rot / 2, step = inter ? 2 : 1, apart = inter ? 1 : rh;
  float inv = 1.f;
  if (qk_norm) {
    float ss = 0.f;
    for (int i = lane; i < dim; i += 32) {                 // a rotation keeps the sum of squares
      const float a = value(i);
      ss += a * a;
    }
    inv = 1.f / sqrtf(warp_sum(ss) / dim + eps);
  }
  if (is_q || slot_ok) {
    T* dst = is_q ? q_out + (static_cast<size_t>(t) * Hq + g) * Dk : k_cache + (static_cast<size_t>(slot) * Hkv + g) * Dk;
    for (int i = lane; i < rh; i += 32) {
      const int a = i * step, b = a + apart;
      const float u = value(a), w = value(b), c = cs[i], s = cs[rh + i];
      put(dst + a, (u * c - w * s) * inv);
      put(dst + b, (w * c + u * s) * inv);
    }
    for (int i = rot + lane; i < dim; i += 32) put(dst + i, value(i) * inv);
    if (is_q)
      for (int i = dim + lane; i < Dk; i += 32) put(dst + i, 0.f);
  }
  shift_state();
}

// The same for rows that can be read four elements at a time (every offset, size and pitch a multiple of 4, `rot` of 8):
// one CTA per token, sixteen lanes per head, all pieces of a head in registers between the norm and the store.
template <typename T, int NP>
__global__ void __launch_bounds__(256)
attn_prep_vec_kernel(const T* __restrict__ proj, long long ld, int off_k, int off_v, const int* __restrict__ positions,
                     const float* __restrict__ cos_sin, const int* __restrict__ slots, const T* __restrict__ v_first,
                     long long ld_first, float lambda, T* __restrict__ q_out, T* __restrict__ k_cache,
                     T* __restrict__ v_cache, int Hq, int Hkv, int dim, int vdim, int Dk, int Dv, int rot, int max_pos,
                     long long num_slots, int qk_norm, float eps) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int t = blockIdx.x, l = threadIdx.x & 15;
  const long long slot = slots[t];
  const bool slot_ok = slot >= 0 && slot < num_slots;
  const T* row = proj + static_cast<size_t>(t) * ld;
  const int pos = min(max(positions[t], 0), max_pos - 1);
  const float* cs = cos_sin + static_cast<size_t>(pos) * rot;
  const int rh = rot / 2;
  const int heads = Hq + 2 * Hkv, groups = blockDim.x >> 4;
  for (int h0 = 0; h0 < heads; h0 += groups) {          // all lanes of a warp stay in the loop (shuffles below)
    const int h = h0 + (threadIdx.x >> 4);
    if (h >= Hq + Hkv) {
      const int g = h - Hq - Hkv;
      if (g < Hkv && slot_ok) {
        const T* v = row + off_v + static_cast<size_t>(g) * vdim;
        const T* f = v_first + static_cast<size_t>(t) * ld_first + static_cast<size_t>(g) * vdim;
        for (int i = 4 * l; i < vdim; i += 64) {
          float4 x = load4(v + i);
          if (v_first != nullptr) {
            const float4 y = load4(f + i);
            const float m = 1.f - lambda;
            x = make_float4(m * x.x + lambda * y.x, m * x.y + lambda * y.y, m * x.z + lambda * y.z, m * x.w + lambda * y.w);
          }
          store4(v_cache + (static_cast<size_t>(slot) * Hkv + g) * Dv + i, x);
        }
      }
    }
    const bool qk = h < Hq + Hkv, is_q = h < Hq;
    const int g = is_q ? h : h - Hq;
    const T* x = row + (is_q ? 0 : off_k) + static_cast<size_t>(g) * dim;
    float4 u[NP], w[NP], r[NP];                           // rotated pairs, dimensions past the rotated ones
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < NP; ++e) {
      const int i = 4 * (l + 16 * e);
      u[e] = w[e] = r[e] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (qk && i < rh) {
        const float4 a = load4(x + i), b = load4(x + rh + i);
        const float4 c = *reinterpret_cast<const float4*>(cs + i), s = *reinterpret_cast<const float4*>(cs + rh + i);
        u[e] = make_float4(a.x * c.x - b.x * s.x, a.y * c.y - b.y * s.y, a.z * c.z - b.z * s.z, a.w * c.w - b.w * s.w);
        w[e] = make_float4(b.x * c.x + a.x * s.x, b.y * c.y + a.y * s.y, b.z * c.z + a.z * s.z, b.w * c.w + a.w * s.w);
      }
      if (qk && rot + i < dim) r[e] = load4(x + rot + i);
      ss += u[e].x * u[e].x + u[e].y * u[e].y + u[e].z * u[e].z + u[e].w * u[e].w + w[e].x * w[e].x + w[e].y * w[e].y +
            w[e].z * w[e].z + w[e].w * w[e].w + r[e].x * r[e].x + r[e].y * r[e].y + r[e].z * r[e].z + r[e].w * r[e].w;
    }
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!qk || (!is_q && !slot_ok)) continue;
    const float inv = qk_norm ? 1.f / sqrtf(ss / dim + eps) : 1.f;
    T* dst = is_q ? q_out + (static_cast<size_t>(t) * Hq + g) * Dk : k_cache + (static_cast<size_t>(slot) * Hkv + g) * Dk;
#pragma unroll
    for (int e = 0; e < NP; ++e) {
      const int i = 4 * (l + 16 * e);
      if (i < rh) {
        store4(dst + i, make_float4(u[e].x * inv, u[e].y * inv, u[e].z * inv, u[e].w * inv));
        store4(dst + rh + i, make_float4(w[e].x * inv, w[e].y * inv, w[e].z * inv, w[e].w * inv));
      }
      if (rot + i < dim) store4(dst + rot + i, make_float4(r[e].x * inv, r[e].y * inv, r[e].z * inv, r[e].w * inv));
    }
    if (is_q)
      for (int i = dim + 4 * l; i < Dk; i += 64) store4(dst + i, make_float4(0.f, 0.f, 0.f, 0.f));
  }
}

// Convolution, interleaved rotation and store of rows that can be read four elements at a time, TAPS <= 8: L lanes per
// (run of `run` consecutive rows, head) with the head's convolution weights in registers, E pieces of 4 L channels.  RB rows
// inside one sequence are loaded together with their TAPS - 1 predecessors (in L1 from the rows before), the first rows of a
// sequence one by one.
template <typename T, int L, int E, int TAPS, int RB>
__global__ void __launch_bounds__(128)
attn_conv_run_kernel(const T* __restrict__ proj, long long ld, int off_k, int off_v, const int* __restrict__ positions,
                     const float* __restrict__ cos_sin, const int* __restrict__ slots, T* __restrict__ q_out,
                     T* __restrict__ k_cache, T* __restrict__ v_cache, int T_, int Hq, int Hkv, int dim, int vdim, int Dk, int Dv,
                     int rot, int max_pos, long long num_slots, int qk_norm, float eps, int run, ConvPast cv) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int l = threadIdx.x % L;
  const int h = blockIdx.y * (blockDim.x / L) + threadIdx.x / L;
  const bool on = h < Hq + 2 * Hkv;                        // lanes past the last head stay for the exchanges
  const int t0 = blockIdx.x * run, t1 = min(T_, t0 + run);
  const bool is_q = h < Hq, is_v = h >= Hq + Hkv;
  const int g = is_q ? h : (is_v ? h - Hq - Hkv : h - Hq), width = is_v ? vdim : dim;
  const int col = (is_q ? 0 : (is_v ? off_v : off_k)) + g * width;
  const int chan = is_v ? (Hq + Hkv) * dim + g * vdim : h * dim;
  const int rh = rot / 2;
  ShortConv<T, TAPS> wt[E];
  bool ok[E];
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = 4 * (l + L * e);
    ok[e] = on && i < width;
    wt[e].weights(cv.w, cv.C, chan + i, ok[e]);
  }
  int b = sequence_of(cv.cu, cv.B, t0), end = cv.cu[b + 1];
  T* st = nullptr;
  const T* old = nullptr;
  auto enter = [&]() {                                     // sequence b: its state, and whether it has a past
    const int n = end - cv.cu[b], slot = cv.slots[b];
    st = slot >= 0 && slot < cv.num_slots ? static_cast<T*>(cv.state) + static_cast<size_t>(slot) * (cv.taps - 1) * cv.C : nullptr;
    old = cv.kv_lens[b] - n > 0 ? st : nullptr;
  };
  enter();
  // where a row goes and its angles: loaded before the row's channels are needed
  struct Target {
    T* dst;                                                // null: nowhere
    float2 c[E], s[E];
  };
  auto target = [&](int t) {
    Target r;
    const long long slot = slots[t];
    const bool to = on && (is_q || (slot >= 0 && slot < num_slots));
    r.dst = !to ? nullptr : is_q ? q_out + (static_cast<size_t>(t) * Hq + g) * Dk
                          : is_v ? v_cache + (static_cast<size_t>(slot) * Hkv + g) * Dv
                                 : k_cache + (static_cast<size_t>(slot) * Hkv + g) * Dk;
    const float* cs = cos_sin + static_cast<size_t>(min(max(positions[t], 0), max_pos - 1)) * rot;
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int i = 4 * (l + L * e);
      r.c[e] = make_float2(1.f, 1.f);
      r.s[e] = make_float2(0.f, 0.f);
      if (to && !is_v && i < rot) {
        r.c[e] = *reinterpret_cast<const float2*>(cs + i / 2);
        r.s[e] = *reinterpret_cast<const float2*>(cs + rh + i / 2);
      }
    }
    return r;
  };
  auto emit = [&](const Target& r, const float4 (&a)[E]) {
    float inv = 1.f;
    if (qk_norm) {                                         // a rotation keeps the sum of squares
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < E; ++e) ss += a[e].x * a[e].x + a[e].y * a[e].y + a[e].z * a[e].z + a[e].w * a[e].w;
#pragma unroll
      for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (!is_v) inv = 1.f / sqrtf(ss / dim + eps);
    }
    if (r.dst == nullptr) return;
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int i = 4 * (l + L * e);
      if (!ok[e]) {
        if (is_q && i < Dk) store4(r.dst + i, make_float4(0.f, 0.f, 0.f, 0.f));
        continue;
      }
      const float4 x = a[e];
      store4(r.dst + i, make_float4((x.x * r.c[e].x - x.y * r.s[e].x) * inv, (x.y * r.c[e].x + x.x * r.s[e].x) * inv,
                                    (x.z * r.c[e].y - x.w * r.s[e].y) * inv, (x.w * r.c[e].y + x.z * r.s[e].y) * inv));
    }
  };
  for (int t = t0; t < t1;) {
    if (t >= end) {
      while (cv.cu[b + 1] <= t) ++b;                       // sequences without tokens in this step are skipped
      end = cv.cu[b + 1];
      enter();
    }
    const int local = t - cv.cu[b];
    const T* row = proj + static_cast<size_t>(t) * ld + col;
    if (RB > 1 && local >= TAPS - 1 && t + RB <= min(t1, end)) {
      float4 x[E][TAPS - 1 + RB];
      Target to[RB];
#pragma unroll
      for (int r = 0; r < RB; ++r) to[r] = target(t + r);
#pragma unroll
      for (int e = 0; e < E; ++e)
#pragma unroll
        for (int j = 0; j < TAPS - 1 + RB; ++j)
          x[e][j] = ok[e] ? load4(row + (j - (TAPS - 1)) * ld + 4 * (l + L * e)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int r = 0; r < RB; ++r) {
        float4 a[E];
#pragma unroll
        for (int e = 0; e < E; ++e) a[e] = wt[e].sum(&x[e][r]);
        emit(to[r], a);
      }
      t += RB;
      continue;
    }
    const Target to = target(t);
    float4 a[E];
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int i = 4 * (l + L * e);
      float4 x[TAPS];
      wt[e].inputs(x, row + i, ld, local, old != nullptr ? old + chan + i : nullptr, cv.C, cv.taps, ok[e]);
      a[e] = wt[e].sum(x);
      // run == 1: these lanes alone read and write these channels' state
      if (cv.update && st != nullptr) wt[e].save(x, st + chan + i, cv.C, cv.taps, ok[e]);
    }
    emit(to, a);
    ++t;
  }
}

// ------------------------------------------------------------------------------------------------
// Paged attention for any head size, fp32 arithmetic.  One warp per (token, query head): each lane scores one key
// of a group of 32, the group's softmax is exchanged by shuffles, and the lanes then split the value dimensions.  Value
// rows are `ldv` elements apart (values that are the first columns of the keys), `sink` has a score per head, `gate` a
// pre-activation per token and head for the output.
// ------------------------------------------------------------------------------------------------
constexpr int kAttnWarps = 4;
constexpr int kMaxOut = 32;        // value dimensions per lane: vdim <= 1024
template <typename T>
struct AnyAttention {
  float scale, softcap;             // softcap 0: scores as they are
  int window, chunk, keep;          // keep: first tokens that stay visible past the window
  const float* sink;                // [Hq] or null
  const T* gate;                    // [T, ld_gate] or null
  long long ld_gate;
};
template <typename T, int NV>
__global__ void __launch_bounds__(kAttnWarps * 32)
attn_any_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                const int* __restrict__ block_tables, const int* __restrict__ cu, const int* __restrict__ kv_lens,
                T* __restrict__ out, int T_, int B, int max_blocks, int bs_shift, int Hq, int Hkv, int Dk, int Dv, int ldv,
                AnyAttention<T> a) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  extern __shared__ float sq[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* qs = sq + warp * Dk;
  const long long job = static_cast<long long>(blockIdx.x) * kAttnWarps + warp;
  if (job >= static_cast<long long>(T_) * Hq) return;
  const int t = static_cast<int>(job / Hq), h = static_cast<int>(job % Hq);
  const int b = sequence_of(cu, B, t);
  const int L = kv_lens[b], n = cu[b + 1] - cu[b];
  const int pos = L - n + (t - cu[b]);
  const int kvh = h / (Hq / Hkv);
  for (int i = lane; i < Dk; i += 32) qs[i] = to_f(q[(static_cast<size_t>(t) * Hq + h) * Dk + i]);
  __syncwarp();
  int lo = a.window > 0 ? pos - a.window + 1 : 0;
  if (a.chunk > 0 && pos > 0) lo = max(lo, pos - pos % a.chunk);
  lo = max(lo, 0);
  float m = a.sink != nullptr ? a.sink[h] : -INFINITY, l = a.sink != nullptr ? 1.f : 0.f;
  float o[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) o[i] = 0.f;
  const int* table = block_tables + static_cast<size_t>(b) * max_blocks;
  // kept first tokens, then the window
  for (int t0 = a.keep > 0 && lo > 0 ? 0 : lo, end = t0 < lo ? min(a.keep, lo) : pos + 1; t0 < end;) {
    const int key = t0 + lane;
    long long row = 0;
    float s = -INFINITY;
    if (key < end) {
      row = (static_cast<long long>(table[key >> bs_shift]) << bs_shift) + (key & ((1 << bs_shift) - 1));
      const T* kp = k_cache + (static_cast<size_t>(row) * Hkv + kvh) * Dk;
      float acc = 0.f;
      int i = 0;
      if (Dk % 4 == 0) {
        float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
        for (; i < Dk; i += 4) {
          const float4 kv = load4(kp + i);
          a0 = fmaf(kv.x, qs[i], a0);
          a1 = fmaf(kv.y, qs[i + 1], a1);
          a2 = fmaf(kv.z, qs[i + 2], a2);
          a3 = fmaf(kv.w, qs[i + 3], a3);
        }
        acc = (a0 + a1) + (a2 + a3);
      }
      for (; i < Dk; ++i) acc = fmaf(to_f(kp[i]), qs[i], acc);
      s = acc * a.scale;
      if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
    }
    float mx = s;
#pragma unroll
    for (int d = 16; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
    const float mn = fmaxf(m, mx);
    const float alpha = expf(m - mn);                 // m = -inf only before the first group: exp(-inf) = 0
    const float pr = expf(s - mn);
    l = l * alpha + warp_sum(pr);
    m = mn;
#pragma unroll
    for (int i = 0; i < NV; ++i) o[i] *= alpha;
    const int cnt = min(32, end - t0);
    for (int j = 0; j < cnt; ++j) {
      const float pj = __shfl_sync(0xffffffffu, pr, j);
      const long long rj = __shfl_sync(0xffffffffu, row, j);
      const T* vp = v_cache + (static_cast<size_t>(rj) * Hkv + kvh) * ldv;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (lane + 32 * i < Dv) o[i] = fmaf(pj, to_f(vp[lane + 32 * i]), o[i]);
    }
    t0 += 32;
    if (t0 >= end && end <= lo) {
      t0 = lo;
      end = pos + 1;
    }
  }
  float inv = l > 0.f ? 1.f / l : 0.f;
  if (a.gate != nullptr) inv *= sigmoid_t<T>(to_f(a.gate[static_cast<size_t>(t) * a.ld_gate + h]));
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (lane + 32 * i < Dv) put(out + (static_cast<size_t>(t) * Hq + h) * Dv + lane + 32 * i, o[i] * inv);
}

// ------------------------------------------------------------------------------------------------
// Inputs of a gated delta rule.  proj[T, ld]: q and k (G heads of dim), v (H of vdim), b (H) at off_q .. off_b;
// a_pre[T, ld_a]: pre-activations of the decays (H x dim, or H).  One warp per (token, unit):
//   units 0 .. G-1            q and k of a head: convolution, SiLU, unit norm (q also times dim^-1/2), and q . k
//   units G .. G+H-1          v of a head: convolution, SiLU; write strength sigmoid(b)
//   units G+H .. G+2H-1       decay exp(-exp(A_log) softplus(a + dt_bias)) of every key channel (one per head: with v)
// q, k and the decays are written with `dimP` columns per head, zero padded.  The convolution reads the previous
// taps - 1 inputs from the step's rows or, before them, from the sequence's state [taps - 1][C] (C = (2 G dim + H vdim)
// channels, oldest first); a sequence that starts at position 0 has zeros there.  With `update` (every sequence
// contributes at most one token) the state is shifted here, otherwise conv_state_kernel does it afterwards.
// ------------------------------------------------------------------------------------------------
struct DeltaPrep {
  long long ld, ld_a;
  int off_q, off_k, off_v, off_b;
  int B, G, H, dim, dimP, vdim, taps, update;
  int head_decay;                 // one decay per head: a_pre [T, H], dt_bias [H], g_out [T, H], written beside beta
};

template <typename T, int NV>
__global__ void __launch_bounds__(256)
delta_prep_kernel(const T* __restrict__ proj, const T* __restrict__ a_pre, const float* __restrict__ conv_t,
                  const float* __restrict__ A_log, const float* __restrict__ dt_bias, const int* __restrict__ cu, const int* __restrict__ kv_lens,
                  const int* __restrict__ state_slots, T* __restrict__ conv_state, float* __restrict__ q_out,
                  float* __restrict__ k_out, float* __restrict__ v_out, float* __restrict__ g_out,
                  float* __restrict__ beta_out, float* __restrict__ qk_out, int T_, int num_slots, DeltaPrep p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int lane = threadIdx.x & 31;
  const int units = p.G + (p.head_decay ? 1 : 2) * p.H;
  const long long job = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (job >= static_cast<long long>(T_) * units) return;
  const int t = static_cast<int>(job / units), u = static_cast<int>(job % units);
  if (u >= p.G + p.H) {
    const int h = u - p.G - p.H;
    const float rate = expf(A_log[h]);
    const T* a = a_pre + static_cast<size_t>(t) * p.ld_a + static_cast<size_t>(h) * p.dim;
    float* g = g_out + (static_cast<size_t>(t) * p.H + h) * p.dimP;
    for (int i = lane; i < p.dimP; i += 32) {
      float v = 0.f;
      if (i < p.dim) {
        const float z = to_f(a[i]) + dt_bias[h * p.dim + i];
        const float sp = z > 20.f ? z : log1pf(expf(z));
        v = expf(-rate * sp);
      }
      g[i] = v;
    }
    return;
  }
  const int b = sequence_of(cu, p.B, t);
  const int n = cu[b + 1] - cu[b], i0 = t - cu[b];
  const int start = kv_lens[b] - n, slot = state_slots[b];
  const int C = 2 * p.G * p.dim + p.H * p.vdim;
  const bool has = slot >= 0 && slot < num_slots;
  T* st = has ? conv_state + static_cast<size_t>(slot) * (p.taps - 1) * C : nullptr;
  T* old = start > 0 ? st : nullptr;                    // null: the sequence starts here, zeros before it
  const bool shift = p.update && has;
  // the lane that convolved channel c (column col) also moves its state by one token
  auto shift_state = [&](int c, int col) {
    for (int j = 0; j + 1 < p.taps - 1; ++j)
      st[static_cast<size_t>(j) * C + c] = old != nullptr ? st[static_cast<size_t>(j + 1) * C + c] : T(0.f);
    if (p.taps > 1) st[static_cast<size_t>(p.taps - 2) * C + c] = proj[static_cast<size_t>(t) * p.ld + col];
  };
  if (u < p.G) {
    float q[NV], k[NV];
    float sq = 0.f, sk = 0.f, dot = 0.f;
#pragma unroll
    for (int e = 0; e < NV; ++e) {
      const int i = lane + 32 * e;
      q[e] = k[e] = 0.f;
      if (i < p.dim) {
        const int c = u * p.dim + i, ck = p.G * p.dim + c;
        q[e] = silu_f(conv_value(proj, p.ld, p.off_q + c, t, i0, conv_t + c, old, C, c, p.taps));
        k[e] = silu_f(conv_value(proj, p.ld, p.off_k + c, t, i0, conv_t + ck, old, C, ck, p.taps));
        if (shift) {
          shift_state(c, p.off_q + c);
          shift_state(ck, p.off_k + c);
        }
        sq += q[e] * q[e];
        sk += k[e] * k[e];
        dot += q[e] * k[e];
      }
    }
    const float iq = 1.f / (sqrtf(warp_sum(sq) + 1e-6f) * sqrtf(static_cast<float>(p.dim)));
    const float ik = 1.f / sqrtf(warp_sum(sk) + 1e-6f);
    dot = warp_sum(dot);
    const size_t o = (static_cast<size_t>(t) * p.G + u) * p.dimP;
#pragma unroll
    for (int e = 0; e < NV; ++e) {
      const int i = lane + 32 * e;
      if (i < p.dimP) {
        q_out[o + i] = q[e] * iq;
        k_out[o + i] = k[e] * ik;
      }
    }
    if (lane == 0) qk_out[static_cast<size_t>(t) * p.G + u] = dot * iq * ik;
    return;
  }
  const int h = u - p.G;
  for (int i = lane; i < p.vdim; i += 32) {
    const int cv = h * p.vdim + i, c = 2 * p.G * p.dim + cv;
    v_out[(static_cast<size_t>(t) * p.H + h) * p.vdim + i] = silu_f(
        conv_value(proj, p.ld, p.off_v + cv, t, i0, conv_t + c, old, C, c, p.taps));
    if (shift) shift_state(c, p.off_v + cv);
  }
  const size_t th = static_cast<size_t>(t) * p.H + h;
  if (lane == 0) beta_out[th] = sigmoid_f(to_f(proj[static_cast<size_t>(t) * p.ld + p.off_b + h]));
  if (p.head_decay && lane == 0)
    g_out[th] = decay_value(to_f(a_pre[static_cast<size_t>(t) * p.ld_a + h]) + dt_bias[h], expf(A_log[h]));
}

// The same for up to TAPS <= 8 taps, with one warp per (run of `run` consecutive rows, unit): the convolution weights
// stay in registers while the warp walks the rows, four channels per lane and piece (E pieces of 128 channels).  RB rows
// inside one sequence are loaded together with their TAPS - 1 predecessors (in L1 from the rows before), the first rows
// of a sequence one by one.  Weights come as [TAPS][C] with absent taps zero.  UNITS: 0 = all units as above, 1 = q and
// k, 2 = v, 3 = decays (prompts: a kernel each, with the registers it needs).
template <typename T, int E, int TAPS, int UNITS, int RB>
__global__ void __launch_bounds__(128)
delta_prep_run_kernel(const T* __restrict__ proj, const T* __restrict__ a_pre, const float* __restrict__ conv_t,
                      const float* __restrict__ A_log, const float* __restrict__ dt_bias, const int* __restrict__ cu,
                      const int* __restrict__ kv_lens, const int* __restrict__ state_slots, T* __restrict__ conv_state,
                      float* __restrict__ q_out, float* __restrict__ k_out, float* __restrict__ v_out,
                      float* __restrict__ g_out, float* __restrict__ beta_out, float* __restrict__ qk_out, int T_,
                      int num_slots, int run, DeltaPrep p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int lane = threadIdx.x & 31;
  const int first = UNITS == 2 ? p.G : (UNITS == 3 ? p.G + p.H : 0);
  const int u = first + blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (u >= (UNITS == 1 ? p.G : (UNITS == 2 || p.head_decay ? p.G + p.H : p.G + 2 * p.H))) return;
  const int t0 = blockIdx.x * run, t1 = min(T_, t0 + run);
  if (UNITS == 3 || (UNITS == 0 && u >= p.G + p.H)) {
    const int h = u - p.G - p.H;
    const float rate = expf(A_log[h]);
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int i = 4 * lane + 128 * e;
      if (i >= p.dimP) continue;
      const bool in = i < p.dim;
      const float4 bias = in ? *reinterpret_cast<const float4*>(dt_bias + h * p.dim + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
      for (int t = t0; t < t1; ++t) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (in) {
          const float4 a = load4(a_pre + static_cast<size_t>(t) * p.ld_a + h * p.dim + i);
          v = make_float4(decay_value(a.x + bias.x, rate), decay_value(a.y + bias.y, rate), decay_value(a.z + bias.z, rate),
                          decay_value(a.w + bias.w, rate));
        }
        store4(g_out + (static_cast<size_t>(t) * p.H + h) * p.dimP + i, v);
      }
    }
    return;
  }
  const int C = 2 * p.G * p.dim + p.H * p.vdim;
  if (UNITS == 3) return;
  const bool is_v = UNITS == 2 || (UNITS == 0 && u >= p.G);
  const int h = is_v ? u - p.G : u, width = is_v ? p.vdim : p.dim;
  // channel and column of the head's first element: q (or v), and k
  const int ca = is_v ? 2 * p.G * p.dim + h * p.vdim : h * p.dim, ck = p.G * p.dim + h * p.dim;
  const int cola = (is_v ? p.off_v + h * p.vdim : p.off_q + h * p.dim), colk = p.off_k + h * p.dim;
  const bool decays = is_v && p.head_decay;
  const float rate_h = decays ? expf(A_log[h]) : 0.f, bias_h = decays ? dt_bias[h] : 0.f;
  ShortConv<T, TAPS> wa[E], wk[E];
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = 4 * lane + 128 * e;
    wa[e].weights(conv_t, C, ca + i, i < width);
    if (!is_v) wk[e].weights(conv_t, C, ck + i, i < width);
  }
  int b = sequence_of(cu, p.B, t0), end = cu[b + 1];
  T* st = nullptr;
  const T* old = nullptr;
  auto enter = [&]() {                             // sequence b: its state, and whether it has a past
    const int n = end - cu[b], slot = state_slots[b];
    st = slot >= 0 && slot < num_slots ? conv_state + static_cast<size_t>(slot) * (p.taps - 1) * C : nullptr;
    old = kv_lens[b] - n > 0 ? st : nullptr;
  };
  enter();
  auto emit = [&](int t, const float4 (&a)[E], const float4 (&k)[E]) {
    if (is_v) {
#pragma unroll
      for (int e = 0; e < E; ++e) {
        const int i = 4 * lane + 128 * e;
        if (i < width) store4(v_out + (static_cast<size_t>(t) * p.H + h) * p.vdim + i, a[e]);
      }
      const size_t th = static_cast<size_t>(t) * p.H + h;
      if (lane == 0) beta_out[th] = sigmoid_f(to_f(proj[static_cast<size_t>(t) * p.ld + p.off_b + h]));
      if (p.head_decay && lane == 1)
        g_out[th] = decay_value(to_f(a_pre[static_cast<size_t>(t) * p.ld_a + h]) + bias_h, rate_h);
      return;
    }
    float sq = 0.f, sk = 0.f, dq = 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e) {
      sq += dot4(a[e], a[e]);
      sk += dot4(k[e], k[e]);
      dq += dot4(a[e], k[e]);
    }
    const float iq = 1.f / (sqrtf(warp_sum(sq) + 1e-6f) * sqrtf(static_cast<float>(p.dim)));
    const float ik = 1.f / sqrtf(warp_sum(sk) + 1e-6f);
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int i = 4 * lane + 128 * e;
      if (i >= p.dimP) continue;
      const size_t o = (static_cast<size_t>(t) * p.G + h) * p.dimP + i;
      store4(q_out + o, make_float4(a[e].x * iq, a[e].y * iq, a[e].z * iq, a[e].w * iq));
      store4(k_out + o, make_float4(k[e].x * ik, k[e].y * ik, k[e].z * ik, k[e].w * ik));
    }
    if (p.update) {                                // only the single-token scan reads q . k
      dq = warp_sum(dq);
      if (lane == 0) qk_out[static_cast<size_t>(t) * p.G + h] = dq * iq * ik;
    }
  };
  for (int t = t0; t < t1;) {
    if (t >= end) {
      while (cu[b + 1] <= t) ++b;                  // sequences without tokens in this step are skipped
      end = cu[b + 1];
      enter();
    }
    const int local = t - cu[b];
    const T* row = proj + static_cast<size_t>(t) * p.ld;
    if (RB > 1 && local >= TAPS - 1 && t + RB <= min(t1, end)) {
      float4 x[E][TAPS - 1 + RB], y[E][TAPS - 1 + RB];
#pragma unroll
      for (int e = 0; e < E; ++e) {
        const int i = 4 * lane + 128 * e;
        const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int j = 0; j < TAPS - 1 + RB; ++j) {
          x[e][j] = i < width ? load4(row + (j - (TAPS - 1)) * p.ld + cola + i) : z;
          y[e][j] = !is_v && i < width ? load4(row + (j - (TAPS - 1)) * p.ld + colk + i) : z;
        }
      }
#pragma unroll
      for (int r = 0; r < RB; ++r) {
        float4 a[E], k[E];
#pragma unroll
        for (int e = 0; e < E; ++e) {
          a[e] = wa[e].apply(&x[e][r]);
          if (!is_v) k[e] = wk[e].apply(&y[e][r]);
        }
        emit(t + r, a, k);
      }
      t += RB;
      continue;
    }
    float4 a[E], k[E];
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int i = 4 * lane + 128 * e;
      const bool ok = i < width;
      float4 x[TAPS], y[TAPS];
      wa[e].inputs(x, row + cola + i, p.ld, local, old != nullptr ? old + ca + i : nullptr, C, p.taps, ok);
      if (!is_v) wk[e].inputs(y, row + colk + i, p.ld, local, old != nullptr ? old + ck + i : nullptr, C, p.taps, ok);
      a[e] = wa[e].apply(x);
      if (!is_v) k[e] = wk[e].apply(y);
      if (p.update && st != nullptr) {             // run == 1: this warp alone reads and writes these channels' state
        wa[e].save(x, st + ca + i, C, p.taps, ok);
        if (!is_v) wk[e].save(y, st + ck + i, C, p.taps, ok);
      }
    }
    emit(t, a, k);
    ++t;
  }
}

// ------------------------------------------------------------------------------------------------
// Prompts with up to four taps and heads of 32, 64 or 128: a CTA convolves 32 rows of 256 neighbouring channels (heads of
// one kind: q, k or v), brought to shared memory with the three rows before them.  A lane owns eight channels of four
// consecutive rows (bound by instructions: 16-byte accesses, packed fp32 multiply-adds).  ATTN: attention inputs as
// attn_conv_run_kernel writes them, otherwise those of a delta rule.  grid (row tiles, channel tiles of q, then k, then v)
// ------------------------------------------------------------------------------------------------
constexpr int kTileRows = 32, kTileCols = 256;
struct ConvTile {
  long long ld;
  int T, off[3], heads[3], width[3];       // of q, k, v
  // attention
  const int *positions, *page_slots;
  const float* cos_sin;
  void *q_out, *k_cache, *v_cache;
  long long num_pages;                     // token slots of the pools
  int rot, max_pos, qk_norm, Dk, Dv;
  float eps;
  // delta rule
  float *q, *k, *v, *g, *beta;
  const void* a_pre;
  long long ld_a;
  const float *A_log, *dt_bias;
  int off_b, head_decay;
};

// eight neighbouring values as four packed pairs
using pair = unsigned long long;
struct Oct {
  pair v[4];
};
__device__ __forceinline__ pair pack_pair(float x, float y) {
  pair r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
  return r;
}
__device__ __forceinline__ float2 unpack_pair(pair p) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(p));
  return r;
}
__device__ __forceinline__ pair fma_pair(pair a, pair b, pair c) {
  pair r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ Oct load8(const float* p) {
  const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(p), b = *reinterpret_cast<const ulonglong2*>(p + 4);
  return Oct{{a.x, a.y, b.x, b.y}};
}
__device__ __forceinline__ Oct load8(const bf16* p) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  auto two = [](uint32_t w) { return pack_pair(__uint_as_float(w << 16), __uint_as_float(w & 0xffff0000u)); };
  return Oct{{two(u.x), two(u.y), two(u.z), two(u.w)}};
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
  store4(p, make_float4(v[0], v[1], v[2], v[3]));
  store4(p + 4, make_float4(v[4], v[5], v[6], v[7]));
}
__device__ __forceinline__ void store8(bf16* p, const float (&v)[8]) {
  uint32_t u[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    u[i] = *reinterpret_cast<const uint32_t*>(&h);
  }
  *reinterpret_cast<uint4*>(p) = make_uint4(u[0], u[1], u[2], u[3]);
}

template <typename T, bool ATTN>
__global__ void __launch_bounds__(256, 2)
conv_tile_kernel(const T* __restrict__ proj, ConvTile p, ConvPast cv) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  constexpr int TAPS = 4, HALO = TAPS - 1, PER = 16 / sizeof(T);      // elements of a 16-byte piece
  using Out = typename std::conditional<ATTN, T, float>::type;
  __shared__ __align__(16) T tile[kTileRows + HALO][kTileCols];
  __shared__ int s_local[kTileRows], s_old[kTileRows];                // place in its sequence; state slot with a past, or -1
  __shared__ int s_row[kTileRows], s_pos[kTileRows];                  // row it is written to (-1: none), position
  const int t0 = blockIdx.x * kTileRows;
  // which channels: kind (0 q, 1 k, 2 v) and first column inside it
  int kind = 0, first = blockIdx.y * kTileCols, chan0 = 0;
  while (kind < 2 && first >= (p.heads[kind] * p.width[kind] + kTileCols - 1) / kTileCols * kTileCols) {
    first -= (p.heads[kind] * p.width[kind] + kTileCols - 1) / kTileCols * kTileCols;
    chan0 += p.heads[kind] * p.width[kind];
    ++kind;
  }
  const int width = p.width[kind], heads = p.heads[kind], cols = min(kTileCols, heads * width - first);
  const T* src = proj + p.off[kind] + first;
  for (int i = threadIdx.x; i < (kTileRows + HALO) * (kTileCols / PER); i += 256) {
    const int r = i / (kTileCols / PER), c = i % (kTileCols / PER) * PER, t = t0 + r - HALO;
    const bool in = t >= 0 && t < p.T && c < cols;
    const uint32_t dst = static_cast<uint32_t>(__cvta_generic_to_shared(&tile[r][c]));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(in ? src + static_cast<size_t>(t) * p.ld + c : src),
                 "r"(in ? 16 : 0)
                 : "memory");
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (threadIdx.x < kTileRows && t0 + threadIdx.x < p.T) {
    const int t = t0 + threadIdx.x, b = sequence_of(cv.cu, cv.B, t), begin = cv.cu[b], slot = cv.slots[b];
    s_local[threadIdx.x] = t - begin;
    s_old[threadIdx.x] = cv.kv_lens[b] - (cv.cu[b + 1] - begin) > 0 && slot >= 0 && slot < cv.num_slots ? slot : -1;
    int row = t;
    if (ATTN) {
      s_pos[threadIdx.x] = min(max(p.positions[t], 0), p.max_pos - 1);
      if (kind > 0) {
        const int page = p.page_slots[t];
        row = page >= 0 && page < p.num_pages ? page : -1;
      }
    }
    s_row[threadIdx.x] = row;
  }
  const int lane = threadIdx.x & 31, c = lane * 8, r0 = (threadIdx.x >> 5) * 4;
  const bool on = c < cols;
  const int chan = chan0 + first + c, h = (first + c) / width, i = (first + c) % width, lanes = width / 8;
  const bool rotate = ATTN && kind < 2 && i < p.rot, normed = kind < 2 && (!ATTN || p.qk_norm);
  const bool scalars = !ATTN && kind == 2 && on && i == 0, decays = scalars && p.head_decay;
  Out* const base = static_cast<Out*>(ATTN ? (kind == 0 ? p.q_out : (kind == 1 ? p.k_cache : p.v_cache))
                                           : static_cast<void*>(kind == 0 ? p.q : (kind == 1 ? p.k : p.v)));
  const int head_pitch = !ATTN ? width : (kind == 2 ? p.Dv : p.Dk);
  Out* const dst0 = base + h * head_pitch + i;
  const size_t pitch = static_cast<size_t>(heads) * head_pitch;
  Oct w[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = on ? load8(cv.w + static_cast<size_t>(j) * cv.C + chan) : Oct{};
  float rate = 0.f, bias = 0.f;
  if (decays) {
    rate = expf(p.A_log[h]);
    bias = p.dt_bias[h];
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  Oct x[4 + HALO];
#pragma unroll
  for (int e = 0; e < 4 + HALO; ++e) x[e] = load8(&tile[r0 + e][c]);
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int t = t0 + r0 + e;
    if (t >= p.T) break;                                              // the same for the whole warp
    const int local = s_local[r0 + e];
    pair acc[4] = {};
    if (local >= HALO) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[q] = fma_pair(w[j].v[q], x[e + j].v[q], acc[q]);
    } else {                                                          // the first rows of a sequence
      const int old = s_old[r0 + e];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const int back = HALO - j, at = cv.taps - 1 + local - back;
        Oct in{};
        if (local >= back) in = x[e + j];
        else if (old >= 0 && at >= 0 && on)
          in = load8(static_cast<const T*>(cv.state) + (static_cast<size_t>(old) * (cv.taps - 1) + at) * cv.C + chan);
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[q] = fma_pair(w[j].v[q], in.v[q], acc[q]);
      }
    }
    float y[8];
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const float2 f = unpack_pair(acc[q]);
      y[2 * q] = ATTN ? f.x : silu_t<T>(f.x);
      y[2 * q + 1] = ATTN ? f.y : silu_t<T>(f.y);
    }
    if (normed) {                                                     // a rotation keeps the sum of squares
      float ss = 0.f;
#pragma unroll
      for (int q = 0; q < 8; ++q) ss = fmaf(y[q], y[q], ss);
      for (int o = lanes / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float inv = ATTN ? rsqrtf(ss / width + p.eps) : rsqrtf(ss + 1e-6f) * (kind == 0 ? rsqrtf(static_cast<float>(width)) : 1.f);
#pragma unroll
      for (int q = 0; q < 8; ++q) y[q] *= inv;
    }
    const int row = s_row[r0 + e];
    if (!on || row < 0) continue;
    if (rotate) {
      const float* cs = p.cos_sin + static_cast<size_t>(s_pos[r0 + e]) * p.rot + i / 2;
      const float4 co = *reinterpret_cast<const float4*>(cs), si = *reinterpret_cast<const float4*>(cs + p.rot / 2);
      const float cf[4] = {co.x, co.y, co.z, co.w}, sf[4] = {si.x, si.y, si.z, si.w};
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float u = y[2 * q], v = y[2 * q + 1];
        y[2 * q] = u * cf[q] - v * sf[q];
        y[2 * q + 1] = v * cf[q] + u * sf[q];
      }
    }
    store8(dst0 + row * pitch, y);
    if (scalars) {
      const size_t th = static_cast<size_t>(t) * heads + h;
      p.beta[th] = sigmoid_f(to_f(proj[static_cast<size_t>(t) * p.ld + p.off_b + h]));
      if (decays) p.g[th] = decay_value(to_f(static_cast<const T*>(p.a_pre)[static_cast<size_t>(t) * p.ld_a + h]) + bias, rate);
    }
  }
}

// shapes conv_tile_kernel takes
template <typename T>
bool conv_tiles(const T* proj, long long ld, const int (&off)[3], int dim, int vdim, int taps, int rot) {
  constexpr int PER = 16 / sizeof(T);
  auto fits = [](int w) { return w == 32 || w == 64 || w == 128; };
  return taps <= 4 && fits(dim) && fits(vdim) && rot % 8 == 0 && ld % PER == 0 && off[0] % PER == 0 && off[1] % PER == 0 && off[2] % PER == 0 &&
         reinterpret_cast<uintptr_t>(proj) % 16 == 0;
}
template <typename T, bool ATTN>
void launch_conv_tiles(const T* proj, const ConvTile& p, const ConvPast& cv, cudaStream_t stream) {
  int tiles = 0;
  for (int i = 0; i < 3; ++i) tiles += (p.heads[i] * p.width[i] + kTileCols - 1) / kTileCols;
  tgi::launch(conv_tile_kernel<T, ATTN>, dim3((p.T + kTileRows - 1) / kTileRows, tiles), dim3(256), 0, stream, proj, p, cv);
}

// ------------------------------------------------------------------------------------------------
// out = RMSNorm(o over `width`) * weight * sigmoid(gate) (SILU: silu(gate)).  o fp32 [T, groups, width]; gate at column `off` of a
// [T, ld] matrix; out rows are `ld_out` wide, columns past groups * width are zeroed by group 0.
// One warp (width <= 1024) or one block per (token, group); grid (tokens, groups / warps of a block).
// ------------------------------------------------------------------------------------------------
template <typename T, bool SILU>
__device__ __forceinline__ float gate_value(float x) {
  if (SILU) return silu_t<T>(x);
  return sigmoid_t<T>(x);
}
template <typename T, bool WARP, bool SILU>
__global__ void __launch_bounds__(256)
gated_norm_kernel(const float* __restrict__ o, const T* __restrict__ gate, long long ld, int off,
                  const float* __restrict__ weight, T* __restrict__ out, long long ld_out, int T_, int groups, int width,
                  float eps) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  __shared__ float red[33];
  const int t = blockIdx.x;
  const int g = WARP ? blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5) : blockIdx.y;
  if (g >= groups) return;                                      // warp- or block-uniform
  const int first = WARP ? (threadIdx.x & 31) : threadIdx.x, step = WARP ? 32 : blockDim.x;
  const float* x = o + (static_cast<size_t>(t) * groups + g) * width;
  const T* gt = gate + static_cast<size_t>(t) * ld + off + static_cast<size_t>(g) * width;
  T* dst = out + static_cast<size_t>(t) * ld_out + static_cast<size_t>(g) * width;
  float ss = 0.f;
  const bool vec = width % 4 == 0 && ld % 4 == 0 && off % 4 == 0 && ld_out % 4 == 0;
  constexpr int NV = WARP ? 2 : 8;                              // pieces per thread kept in registers
  if (vec && width <= NV * 4 * step) {
    float4 v[NV];
#pragma unroll
    for (int e = 0; e < NV; ++e) {
      const int i = (first + e * step) * 4;
      v[e] = i < width ? load4(x + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += dot4(v[e], v[e]);
    }
    ss = WARP ? warp_sum(ss) : block_sum(ss, red);
    const float inv = 1.f / sqrtf(ss / width + eps);
#pragma unroll
    for (int e = 0; e < NV; ++e) {
      const int i = (first + e * step) * 4;
      if (i < width) {
        const float4 w = load4(weight + i), s = load4(gt + i);
        store4(dst + i, make_float4(v[e].x * inv * w.x * gate_value<T, SILU>(s.x), v[e].y * inv * w.y * gate_value<T, SILU>(s.y),
                                    v[e].z * inv * w.z * gate_value<T, SILU>(s.z), v[e].w * inv * w.w * gate_value<T, SILU>(s.w)));
      }
    }
    if (g == 0)
      for (int i = groups * width + first; i < ld_out; i += step) put(out + static_cast<size_t>(t) * ld_out + i, 0.f);
    return;
  }
  if (vec) {
    for (int i = first * 4; i < width; i += step * 4) {
      const float4 v = load4(x + i);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int i = first; i < width; i += step) ss += x[i] * x[i];
  }
  ss = WARP ? warp_sum(ss) : block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / width + eps);
  if (vec) {
    for (int i = first * 4; i < width; i += step * 4) {
      const float4 v = load4(x + i), w = load4(weight + i), s = load4(gt + i);
      store4(dst + i, make_float4(v.x * inv * w.x * gate_value<T, SILU>(s.x), v.y * inv * w.y * gate_value<T, SILU>(s.y),
                                  v.z * inv * w.z * gate_value<T, SILU>(s.z), v.w * inv * w.w * gate_value<T, SILU>(s.w)));
    }
  } else {
    for (int i = first; i < width; i += step) put(dst + i, x[i] * inv * weight[i] * gate_value<float, SILU>(to_f(gt[i])));
  }
  if (g == 0)
    for (int i = groups * width + first; i < ld_out; i += step) put(out + static_cast<size_t>(t) * ld_out + i, 0.f);
}

int done() { return cudaGetLastError() == cudaSuccess ? 0 : -3; }

template <typename T>
int residual_norm(const void* d1, const void* d2, const float* residual, const int* rows, const void* w1, const void* w2,
                  const void* b1, void* o1, void* o2, float* res_out, int n, int H, int layer, float eps, float scale,
                  float offset, cudaStream_t stream) {
  const ResidualNorm<T> p{static_cast<const T*>(d1), static_cast<const T*>(d2), residual, rows, static_cast<const T*>(w1),
                          static_cast<const T*>(w2), static_cast<const T*>(b1), static_cast<T*>(o1), static_cast<T*>(o2),
                          res_out, H, layer, eps, scale, offset};
  if (H % 4 == 0 && H / 4 <= 4 * 1024) {
    const int vecs = H / 4;
    int threads = vecs >= 1024 ? 512 : ((vecs + 31) / 32) * 32;
    if (threads > 256 && vecs <= 1024) threads = 256;
    const int vpt = (vecs + threads - 1) / threads;
    auto go = [&](auto kern) { tgi::launch(kern, dim3(n), dim3(threads), 0, stream, p); };
    if (vpt <= 1) go(residual_norm_kernel<T, 1>);
    else if (vpt <= 2) go(residual_norm_kernel<T, 2>);
    else if (vpt <= 4) go(residual_norm_kernel<T, 4>);
    else go(residual_norm_kernel<T, 8>);
  } else {
    tgi::launch(residual_norm_kernel<T, 0>, dim3(n), dim3(256), 0, stream, p);
  }
  return done();
}

template <typename T>
int attn_any(const void* q, const void* k, const void* v, const int* bt, const int* cu, const int* kv, void* out, int T_,
             int B, int max_blocks, int bs_shift, int Hq, int Hkv, int Dk, int Dv, int ldv, const AnyAttention<T>& a,
             cudaStream_t stream) {
  const long long jobs = static_cast<long long>(T_) * Hq;
  const dim3 grid(static_cast<unsigned>((jobs + kAttnWarps - 1) / kAttnWarps)), block(kAttnWarps * 32);
  const size_t smem = static_cast<size_t>(kAttnWarps) * Dk * sizeof(float);
  if (smem > 48 * 1024 || Dv > 32 * kMaxOut) return -12;
  auto go = [&](auto kern) {
    tgi::launch(kern, grid, block, smem, stream, static_cast<const T*>(q), static_cast<const T*>(k), static_cast<const T*>(v),
                bt, cu, kv, static_cast<T*>(out), T_, B, max_blocks, bs_shift, Hq, Hkv, Dk, Dv, ldv, a);
    return done();
  };
  if (Dv <= 64) return go(attn_any_kernel<T, 2>);
  if (Dv <= 128) return go(attn_any_kernel<T, 4>);
  if (Dv <= 256) return go(attn_any_kernel<T, 8>);
  if (Dv <= 512) return go(attn_any_kernel<T, 16>);
  return go(attn_any_kernel<T, kMaxOut>);
}

template <typename T>
int delta_prep(const void* proj, const void* a_pre, const float* conv_t, const float* A_log, const float* dt_bias,
               const int* cu, const int* kv, const int* slots, void* conv_state, float* q, float* k, float* v, float* g,
               float* beta, float* qk, int T_, int num_slots, const DeltaPrep& p, cudaStream_t stream) {
  const T* x = static_cast<const T*>(proj);
  const T* a = static_cast<const T*>(a_pre);
  T* st = static_cast<T*>(conv_state);
  const int units = p.G + (p.head_decay ? 1 : 2) * p.H, C = 2 * p.G * p.dim + p.H * p.vdim;
  const bool vec = p.taps <= 8 && p.dim % 4 == 0 && p.vdim % 4 == 0 && p.vdim <= 256 && p.ld % 4 == 0 &&
                   p.off_q % 4 == 0 && p.off_k % 4 == 0 && p.off_v % 4 == 0 &&
                   reinterpret_cast<uintptr_t>(proj) % (4 * sizeof(T)) == 0 &&
                   (p.head_decay || (p.ld_a % 4 == 0 && reinterpret_cast<uintptr_t>(a_pre) % (4 * sizeof(T)) == 0));
  if (vec) {
    const bool one = p.dimP <= 128 && p.vdim <= 128;
    auto go = [&](auto kern, int count, int run) {
      tgi::launch(kern, dim3((T_ + run - 1) / run, (count + 3) / 4), dim3(128), 0, stream, x, a, conv_t, A_log, dt_bias, cu, kv,
                  slots, st, q, k, v, g, beta, qk, T_, num_slots, run, p);
    };
    if (p.update) {
      if (p.taps <= 4) one ? go(delta_prep_run_kernel<T, 1, 4, 0, 1>, units, 1) : go(delta_prep_run_kernel<T, 2, 4, 0, 1>, units, 1);
      else one ? go(delta_prep_run_kernel<T, 1, 8, 0, 1>, units, 1) : go(delta_prep_run_kernel<T, 2, 8, 0, 1>, units, 1);
    } else if (p.dimP == p.dim && conv_tiles<T>(x, p.ld, {p.off_q, p.off_k, p.off_v}, p.dim, p.vdim, p.taps, 0)) {
      ConvTile c{};
      c.ld = p.ld; c.T = T_; c.off_b = p.off_b; c.head_decay = p.head_decay;
      c.off[0] = p.off_q; c.off[1] = p.off_k; c.off[2] = p.off_v;
      c.heads[0] = c.heads[1] = p.G; c.heads[2] = p.H;
      c.width[0] = c.width[1] = p.dim; c.width[2] = p.vdim;
      c.q = q; c.k = k; c.v = v; c.g = g; c.beta = beta;
      c.a_pre = a_pre; c.ld_a = p.ld_a; c.A_log = A_log; c.dt_bias = dt_bias;
      launch_conv_tiles<T, false>(x, c, ConvPast{conv_t, cu, kv, slots, conv_state, p.B, p.taps, C, num_slots, 0}, stream);
      if (!p.head_decay) go(delta_prep_run_kernel<T, 1, 4, 3, 1>, p.H, 16);
    } else if (p.taps <= 4 && one) {
      go(delta_prep_run_kernel<T, 1, 4, 1, 2>, p.G, 16);
      go(delta_prep_run_kernel<T, 1, 4, 2, 4>, p.H, 32);
      if (!p.head_decay) go(delta_prep_run_kernel<T, 1, 4, 3, 1>, p.H, 16);
    } else if (p.taps <= 4) {
      go(delta_prep_run_kernel<T, 2, 4, 0, 1>, units, 16);
    } else {
      one ? go(delta_prep_run_kernel<T, 1, 8, 0, 1>, units, 16) : go(delta_prep_run_kernel<T, 2, 8, 0, 1>, units, 16);
    }
  } else {
    const float* first = conv_t + static_cast<size_t>(delta_tap_rows(p.taps) - p.taps) * C;
    const long long jobs = static_cast<long long>(T_) * units;
    const dim3 grid(static_cast<unsigned>((jobs + 7) / 8));
    auto go = [&](auto kern) {
      tgi::launch(kern, grid, dim3(256), 0, stream, x, a, first, A_log, dt_bias, cu, kv, slots, st, q, k, v, g, beta, qk, T_,
                  num_slots, p);
    };
    if (p.dimP <= 64) go(delta_prep_kernel<T, 2>);
    else if (p.dimP <= 128) go(delta_prep_kernel<T, 4>);
    else go(delta_prep_kernel<T, 8>);
  }
  if (!p.update && p.taps > 1)
    tgi::launch(conv_state_kernel<T>, dim3((C + 255) / 256, p.B), dim3(256), 0, stream, x, p.ld, p.G * p.dim, p.G * p.dim,
                p.off_q, p.off_k, p.off_v, ConvPast{nullptr, cu, kv, slots, conv_state, p.B, p.taps, C, num_slots, 0});
  return done();
}

template <typename T>
int gated_norm(const float* o, const void* gate, long long ld, int off, const float* w, void* out, long long ld_out, int T_,
               int groups, int width, float eps, int silu, cudaStream_t stream) {
  auto go = [&](auto kern, dim3 grid, int threads) {
    tgi::launch(kern, grid, dim3(threads), 0, stream, o, static_cast<const T*>(gate), ld, off, w, static_cast<T*>(out), ld_out,
                T_, groups, width, eps);
  };
  if (width <= 1024) {
    const int warps = groups < 8 ? groups : 8;
    const dim3 grid(T_, (groups + warps - 1) / warps);
    silu ? go(gated_norm_kernel<T, true, true>, grid, 32 * warps) : go(gated_norm_kernel<T, true, false>, grid, 32 * warps);
  } else {
    const dim3 grid(T_, groups);
    silu ? go(gated_norm_kernel<T, false, true>, grid, 256) : go(gated_norm_kernel<T, false, false>, grid, 256);
  }
  return done();
}

}  // namespace

// `f32` selects the build: 1 = fp32 activations, weights and pages, 0 = bf16.
extern "C" {

// d2, w2 (with o2), b1 and rows may be null; d1 null: the stream as it is.  layer: LayerNorm instead of RMSNorm
int tgi_residual_norm(int f32, const void* d1, const void* d2, const float* residual, const int* rows, const void* w1,
                      const void* w2, const void* b1, void* o1, void* o2, float* res_out, int n, int H, int layer, float eps,
                      float scale, float offset, cudaStream_t stream) {
  if (n <= 0) return 0;
  return f32 ? residual_norm<float>(d1, d2, residual, rows, w1, w2, b1, o1, o2, res_out, n, H, layer, eps, scale, offset, stream)
             : residual_norm<bf16>(d1, d2, residual, rows, w1, w2, b1, o1, o2, res_out, n, H, layer, eps, scale, offset, stream);
}

int tgi_embed_residual(int f32, const int* ids, const void* table, float* out, int T, int H, int vocab, float scale,
                       cudaStream_t stream) {
  if (T <= 0) return 0;
  if (f32) tgi::launch(embed_residual_kernel<float>, dim3(T), dim3(256), 0, stream, ids, static_cast<const float*>(table), out, H, vocab, scale);
  else tgi::launch(embed_residual_kernel<bf16>, dim3(T), dim3(256), 0, stream, ids, static_cast<const bf16*>(table), out, H, vocab, scale);
  return done();
}

int tgi_activation(int f32, const void* in, void* out, long long n, int act, cudaStream_t stream) {
  if (n <= 0) return 0;
  long long blocks = (n / 4 + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (blocks < 1) blocks = 1;
  const dim3 grid(static_cast<unsigned>(blocks));
  if (f32) tgi::launch(activation_kernel<float>, grid, dim3(256), 0, stream, static_cast<const float*>(in), static_cast<float*>(out), n, act);
  else tgi::launch(activation_kernel<bf16>, grid, dim3(256), 0, stream, static_cast<const bf16*>(in), static_cast<bf16*>(out), n, act);
  return done();
}

// in [T, 2 I] (gate, up) -> out [T, I] = act(gate) * up
int tgi_act_mul_any(int f32, const void* in, void* out, int T, int I, int act, cudaStream_t stream) {
  const long long n = static_cast<long long>(T) * I;
  if (n <= 0) return 0;
  const dim3 grid(static_cast<unsigned>((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16));
  if (f32) tgi::launch(act_mul_any_kernel<float>, grid, dim3(256), 0, stream, static_cast<const float*>(in), static_cast<float*>(out), n, I, act);
  else tgi::launch(act_mul_any_kernel<bf16>, grid, dim3(256), 0, stream, static_cast<const bf16*>(in), static_cast<bf16*>(out), n, I, act);
  return done();
}

// `conv_t` (optional): weights [tgi_delta_tap_rows(taps)][C] of short convolutions on q, k and v, with the sequences' past
// inputs in conv_state [conv_slots][taps - 1][C]; `update`: no sequence brings more than one token.  `inter`: rotate pairs
// 2i, 2i + 1.
int tgi_attn_prep(int f32, const void* proj, long long ld, int off_k, int off_v, const int* positions, const float* cos_sin,
                  const int* slots, const void* v_first, long long ld_first, float lambda, void* q_out, void* k_cache,
                  void* v_cache, int T, int Hq, int Hkv, int dim, int vdim, int Dk, int Dv, int rot, int max_pos,
                  long long num_slots, int qk_norm, float eps, int inter, const float* conv_t, const int* cu,
                  const int* kv_lens, const int* state_slots, void* conv_state, int B, int taps, int conv_slots, int update,
                  cudaStream_t stream) {
  if (T <= 0) return 0;
  if (rot % 2 != 0 || rot > dim || Dk < dim || Dv < vdim) return -10;
  const bool conv = conv_t != nullptr;
  if (conv && (taps < 1 || B < 1 || B > 65535)) return -10;
  ConvPast cv{conv_t, cu, kv_lens, state_slots, conv_state, B, taps, (Hq + Hkv) * dim + Hkv * vdim, conv_slots, update};
  const bool quads = ld % 4 == 0 && off_k % 4 == 0 && off_v % 4 == 0 && dim % 4 == 0 && vdim % 4 == 0 && Dk % 4 == 0 &&
                     Dv % 4 == 0 && dim <= 256 && reinterpret_cast<uintptr_t>(proj) % (f32 ? 16 : 8) == 0;
  auto finish = [&]() {                                    // the state of sequences that brought several tokens
    if (conv && !update && taps > 1) {
      const dim3 grid((cv.C + 255) / 256, B);
      if (f32) tgi::launch(conv_state_kernel<float>, grid, dim3(256), 0, stream, static_cast<const float*>(proj), ld, Hq * dim, Hkv * dim, 0, off_k, off_v, cv);
      else tgi::launch(conv_state_kernel<bf16>, grid, dim3(256), 0, stream, static_cast<const bf16*>(proj), ld, Hq * dim, Hkv * dim, 0, off_k, off_v, cv);
    }
    return done();
  };
  if (conv && inter && quads && rot % 4 == 0 && v_first == nullptr && taps <= 8 && vdim <= 256 && Dk <= 256) {
    auto go = [&](auto kern, auto tag, int lanes, int run) {
      using E = decltype(tag);
      const int per = 128 / lanes;
      tgi::launch(kern, dim3((T + run - 1) / run, (Hq + 2 * Hkv + per - 1) / per), dim3(128), 0, stream,
                  static_cast<const E*>(proj), ld, off_k, off_v, positions, cos_sin, slots, static_cast<E*>(q_out),
                  static_cast<E*>(k_cache), static_cast<E*>(v_cache), T, Hq, Hkv, dim, vdim, Dk, Dv, rot, max_pos, num_slots,
                  qk_norm, eps, run, cv);
    };
    auto shape = [&](auto tag) {
      using E = decltype(tag);
      const E* x = static_cast<const E*>(proj);
      if (!update && Dk == dim && Dv % 8 == 0 && num_slots < (1ll << 31) && conv_tiles<E>(x, ld, {0, off_k, off_v}, dim, vdim, taps, rot)) {
        ConvTile c{};
        c.ld = ld; c.T = T;
        c.off[1] = off_k; c.off[2] = off_v;
        c.heads[0] = Hq; c.heads[1] = c.heads[2] = Hkv;
        c.width[0] = c.width[1] = dim; c.width[2] = vdim;
        c.positions = positions; c.page_slots = slots; c.cos_sin = cos_sin;
        c.q_out = q_out; c.k_cache = k_cache; c.v_cache = v_cache; c.num_pages = num_slots;
        c.rot = rot; c.max_pos = max_pos; c.qk_norm = qk_norm; c.Dk = Dk; c.Dv = Dv; c.eps = eps;
        launch_conv_tiles<E, true>(x, c, cv, stream);
        return;
      }
      const int w = Dk > vdim ? Dk : vdim;                 // the columns past `dim` of q_out are written too
      if (taps <= 4) {
        if (update) {
          if (w <= 64) go(attn_conv_run_kernel<E, 16, 1, 4, 1>, tag, 16, 1);
          else if (w <= 128) go(attn_conv_run_kernel<E, 32, 1, 4, 1>, tag, 32, 1);
          else go(attn_conv_run_kernel<E, 32, 2, 4, 1>, tag, 32, 1);
        } else {
          if (w <= 64) go(attn_conv_run_kernel<E, 16, 1, 4, 4>, tag, 16, 16);
          else if (w <= 128) go(attn_conv_run_kernel<E, 32, 1, 4, 4>, tag, 32, 16);
          else go(attn_conv_run_kernel<E, 32, 2, 4, 2>, tag, 32, 16);
        }
      } else {
        if (w <= 128) go(attn_conv_run_kernel<E, 32, 1, 8, 1>, tag, 32, update ? 1 : 16);
        else go(attn_conv_run_kernel<E, 32, 2, 8, 1>, tag, 32, update ? 1 : 16);
      }
    };
    if (f32) shape(float());
    else shape(bf16());
    return finish();
  }
  const bool vec = !conv && !inter && quads && rot % 8 == 0 && ld_first % 4 == 0 &&
                   reinterpret_cast<uintptr_t>(v_first) % (f32 ? 16 : 8) == 0;
  if (vec) {
    auto go = [&](auto kern, auto tag) {
      using E = decltype(tag);
      tgi::launch(kern, dim3(T), dim3(256), 0, stream, static_cast<const E*>(proj), ld, off_k, off_v, positions, cos_sin,
                  slots, static_cast<const E*>(v_first), ld_first, lambda, static_cast<E*>(q_out), static_cast<E*>(k_cache),
                  static_cast<E*>(v_cache), Hq, Hkv, dim, vdim, Dk, Dv, rot, max_pos, num_slots, qk_norm, eps);
      return done();
    };
    // pieces per lane: rotated halves and the rest are each at most NP x 64 elements
    const int np = (max(rot / 2, dim - rot) + 63) / 64;
    if (np <= 1) return f32 ? go(attn_prep_vec_kernel<float, 1>, float()) : go(attn_prep_vec_kernel<bf16, 1>, bf16());
    if (np <= 2) return f32 ? go(attn_prep_vec_kernel<float, 2>, float()) : go(attn_prep_vec_kernel<bf16, 2>, bf16());
    return f32 ? go(attn_prep_vec_kernel<float, 4>, float()) : go(attn_prep_vec_kernel<bf16, 4>, bf16());
  }
  const long long jobs = static_cast<long long>(T) * (Hq + 2 * Hkv);
  const dim3 grid(static_cast<unsigned>((jobs + 7) / 8));
  if (conv) cv.w += static_cast<size_t>(delta_tap_rows(taps) - taps) * cv.C;
  auto go = [&](auto kern, auto tag) {
    using E = decltype(tag);
    tgi::launch(kern, grid, dim3(256), 0, stream, static_cast<const E*>(proj), ld, off_k, off_v, positions, cos_sin, slots,
                static_cast<const E*>(v_first), ld_first, lambda, static_cast<E*>(q_out), static_cast<E*>(k_cache),
                static_cast<E*>(v_cache), T, Hq, Hkv, dim, vdim, Dk, Dv, rot, max_pos, num_slots,
                qk_norm, eps, inter, cv);
  };
  if (f32) go(attn_prep_kernel<float>, float());
  else go(attn_prep_kernel<bf16>, bf16());
  return finish();
}

// Value rows are `ldv` elements apart.  `sink` (optional): a score per head; `gate` (optional, [T, ld_gate]): the output of
// head h is multiplied by the sigmoid of its column h.
int tgi_attn_any(int f32, const void* q, const void* k_cache, const void* v_cache, const int* block_tables, const int* cu,
                 const int* kv_lens, void* out, int T, int B, int max_blocks, int block_size, int Hq, int Hkv, int Dk, int Dv,
                 int ldv, float scale, float softcap, int window, int chunk, int keep, const float* sink, const void* gate,
                 long long ld_gate, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (Hq % Hkv != 0 || block_size <= 0 || (block_size & (block_size - 1)) != 0) return -10;
  int shift = 0;
  while ((1 << shift) < block_size) ++shift;
  return f32 ? attn_any<float>(q, k_cache, v_cache, block_tables, cu, kv_lens, out, T, B, max_blocks, shift, Hq, Hkv, Dk, Dv, ldv,
                               {scale, softcap, window, chunk, keep, sink, static_cast<const float*>(gate), ld_gate}, stream)
             : attn_any<bf16>(q, k_cache, v_cache, block_tables, cu, kv_lens, out, T, B, max_blocks, shift, Hq, Hkv, Dk, Dv, ldv,
                              {scale, softcap, window, chunk, keep, sink, static_cast<const bf16*>(gate), ld_gate}, stream);
}

// Rows of the [rows][channels] convolution weights tgi_delta_prep wants for `taps` taps (the first rows are zero).
int tgi_delta_tap_rows(int taps) { return delta_tap_rows(taps); }

int tgi_delta_prep(int f32, const void* proj, long long ld, int off_q, int off_k, int off_v, int off_b, const void* a_pre,
                   long long ld_a, const float* conv_t, const float* A_log, const float* dt_bias, const int* cu,
                   const int* kv_lens, const int* state_slots, void* conv_state, float* q, float* k, float* v, float* g,
                   float* beta, float* qk, int T, int B, int num_slots, int G, int H, int dim, int dimP, int vdim, int taps,
                   int update, int head_decay, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (H % G != 0 || dimP < dim || dimP > 256 || taps < 1 || B > 65535) return -10;
  const DeltaPrep p{ld, ld_a, off_q, off_k, off_v, off_b, B, G, H, dim, dimP, vdim, taps, update, head_decay};
  return f32 ? delta_prep<float>(proj, a_pre, conv_t, A_log, dt_bias, cu, kv_lens, state_slots, conv_state, q, k, v, g, beta,
                                 qk, T, num_slots, p, stream)
             : delta_prep<bf16>(proj, a_pre, conv_t, A_log, dt_bias, cu, kv_lens, state_slots, conv_state, q, k, v, g, beta, qk,
                                T, num_slots, p, stream);
}

int tgi_gated_norm(int f32, const float* o, const void* gate, long long ld, int off, const float* weight, void* out,
                   long long ld_out, int T, int groups, int width, float eps, int silu, cudaStream_t stream) {
  if (T <= 0) return 0;
  return f32 ? gated_norm<float>(o, gate, ld, off, weight, out, ld_out, T, groups, width, eps, silu, stream)
             : gated_norm<bf16>(o, gate, ld, off, weight, out, ld_out, T, groups, width, eps, silu, stream);
}

}  // extern "C"
