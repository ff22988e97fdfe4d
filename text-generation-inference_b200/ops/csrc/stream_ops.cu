// Steps of an fp32 residual stream whose blocks are normed on the way in and on the way out, in a bf16 and an fp32 build of
// the activations:
//   stream step         norm of a block's output, addition to the stream, weighted sum over the stream and the results of
//                       earlier layers, norm for the next block and, in steps of single tokens, its input convolution
//   input convolution   causal convolution over time of every channel that a mixer reads, with the sequences' last inputs
//                       as state
// Sums, norms and the stream are fp32 in both builds.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <type_traits>

#include "launch.cuh"
#include "mixer_util.cuh"

namespace {

using namespace mixer;

constexpr int kMaxTaps = 8;       // of the vector kernels

// Convolution over time: a sequence's previous taps - 1 inputs come from the step's rows or, before them, from its state
// [taps - 1][H], oldest first; a sequence that starts at position 0 has zeros there.
struct InputConv {
  const float* w;                 // [taps][H], oldest input first; null: no convolution
  const int *cu, *kv_lens, *slots;
  void* state;                    // [num_slots][taps - 1][H]
  int B, taps, num_slots;
};

// ------------------------------------------------------------------------------------------------
// new = residual + RMSNorm(delta) * post (post null: + delta; delta null: residual as it is)
// r = new, or (depth) sum_{j < index} dw[j] streams[j] + dw[index] new, with new kept as streams[index] (keep)
// out = RMSNorm(r) * w * gain, then (conv, one token per sequence) convolved, the state shifted by one token
// One CTA per output row; `rows` (optional) picks the input row.  VPT float4 per thread stay in registers; VPT == 0: any width,
// the row in shared memory.
// ------------------------------------------------------------------------------------------------
template <typename T>
struct StreamStep {
  const T *delta, *post, *w;
  const float* residual;
  const int* rows;
  float* streams;                 // [index + 1 ..][n][H] or null
  const float* dw;                // [index + 1]
  long long pitch;                // floats from a stream to the next
  T* out;
  float* res_out;                 // null: r is not kept
  int H, index, keep;
  float eps, gain;
  InputConv conv;
};

// state of the sequence that brings row t, and whether it holds anything yet
template <typename T>
__device__ __forceinline__ T* conv_slot(const InputConv& c, int t, int H, bool& fresh) {
  const int b = sequence_of(c.cu, c.B, t), n = c.cu[b + 1] - c.cu[b], slot = c.slots[b];
  fresh = c.kv_lens[b] - n <= 0;
  return slot >= 0 && slot < c.num_slots ? static_cast<T*>(c.state) + static_cast<size_t>(slot) * (c.taps - 1) * H : nullptr;
}

// four elements as they lie in memory: loaded early, converted when they are needed
template <typename T>
struct Quad;
template <>
struct Quad<float> {
  using type = float4;
  static __device__ __forceinline__ float4 value(float4 v) { return v; }
};
template <>
struct Quad<bf16> {
  using type = uint2;
  static __device__ __forceinline__ float4 value(uint2 u) { return load4(reinterpret_cast<const bf16*>(&u)); }
};
// sum over the block with one barrier; `red` holds one float per warp and is used for one sum only
__device__ __forceinline__ float block_sum_once(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) t += red[w];
  return t;
}
__device__ __forceinline__ float4 fma4(float f, float4 a, float4 b) {
  return make_float4(fmaf(f, a.x, b.x), fmaf(f, a.y, b.y), fmaf(f, a.z, b.z), fmaf(f, a.w, b.w));
}
__device__ __forceinline__ float4 fma4(float4 f, float4 a, float4 b) {
  return make_float4(fmaf(f.x, a.x, b.x), fmaf(f.y, a.y, b.y), fmaf(f.z, a.z, b.z), fmaf(f.w, a.w, b.w));
}
__device__ __forceinline__ float square4(float4 a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }

// CONV: most taps of the input convolution, 0: there is none.  AVG: with the weighted sum (VPT > 0).  A step of single tokens
// waits for latencies, so all it reads is asked for at the start; a prompt's steps want many rows in flight: two blocks of 512
// threads per SM, 8192 x 4096: 93 / 197 us (without / with a sum of five), 168 / 296 with one.
template <typename T, int VPT, int CONV, bool AVG>
__global__ void __launch_bounds__(CONV > 0 ? 1024 : 512, CONV > 0 ? 1 : 2)
stream_step_kernel(const StreamStep<T> p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  __shared__ float red[2][33];
  extern __shared__ float held[];                          // VPT == 0: [H]
  const int row = p.rows != nullptr ? p.rows[blockIdx.x] : blockIdx.x, H = p.H;
  const size_t in = static_cast<size_t>(row) * H, ob = static_cast<size_t>(blockIdx.x) * H;
  T* st = nullptr;
  bool fresh = true;
  if constexpr (VPT > 0) {
    using Raw = typename Quad<T>::type;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    auto col = [&](int i) { return static_cast<int>(threadIdx.x + i * blockDim.x) * 4; };
    auto raw = [&](const T* src) { return *reinterpret_cast<const Raw*>(src); };
    // everything a column needs is on its way before the first sum
    float4 x[VPT];
    Raw d[VPT], post[VPT], w[VPT], past[CONV > 1 ? VPT : 1][CONV > 1 ? CONV - 1 : 1];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = col(i);
      if (c < H) {
        x[i] = *reinterpret_cast<const float4*>(p.residual + in + c);
        if (p.delta != nullptr) d[i] = raw(p.delta + in + c);
        if constexpr (CONV > 0) {
          w[i] = raw(p.w + c);
          if (p.post != nullptr) post[i] = raw(p.post + c);
          for (int j = 0; j < p.conv.taps; ++j)            // wanted last
            asm volatile("prefetch.global.L2 [%0];" ::"l"(p.conv.w + static_cast<size_t>(j) * H + c));
        }
      }
    }
    if constexpr (CONV > 0) {
      st = conv_slot<T>(p.conv, row, H, fresh);
      if constexpr (CONV > 1) {
        if (st != nullptr && !fresh) {
#pragma unroll
          for (int i = 0; i < VPT; ++i) {
#pragma unroll
            for (int j = 0; j < CONV - 1; ++j)
              if (j < p.conv.taps - 1 && col(i) < H) past[i][j] = raw(st + static_cast<size_t>(j) * H + col(i));
          }
        }
      }
    }
    float4 sum[AVG ? VPT : 1];
    if constexpr (AVG) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = col(i);
        sum[i] = zero;
        if (c < H) {
          const float* src = p.streams + in + c;
#pragma unroll 4
          for (int j = 0; j < p.index; ++j) sum[i] = fma4(p.dw[j], *reinterpret_cast<const float4*>(src + j * p.pitch), sum[i]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = col(i);
      if (c < H && p.delta != nullptr) ss += square4(Quad<T>::value(d[i]));
    }
    if (p.delta != nullptr) {
      const float inv = p.post != nullptr ? 1.f / sqrtf(block_sum_once(ss, red[0]) / H + p.eps) : 1.f;
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        if (col(i) >= H) continue;
        float4 v = Quad<T>::value(d[i]);
        if (p.post != nullptr) {
          v = make_float4(v.x * inv, v.y * inv, v.z * inv, v.w * inv);
          x[i] = fma4(v, Quad<T>::value(CONV > 0 ? post[i] : raw(p.post + col(i))), x[i]);
        } else {
          x[i] = make_float4(x[i].x + v.x, x[i].y + v.y, x[i].z + v.z, x[i].w + v.w);
        }
      }
    }
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = col(i);
      if (c >= H) continue;
      if constexpr (AVG) {
        if (p.keep) store4(p.streams + p.index * p.pitch + in + c, x[i]);
        x[i] = fma4(p.dw[p.index], x[i], sum[i]);
      }
      if (p.res_out != nullptr) store4(p.res_out + ob + c, x[i]);
      ss += square4(x[i]);
    }
    const float inv = p.gain / sqrtf(block_sum_once(ss, red[1]) / H + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = col(i);
      if (c >= H) continue;
      const float4 g = Quad<T>::value(CONV > 0 ? w[i] : raw(p.w + c));
      float4 y = make_float4(x[i].x * inv * g.x, x[i].y * inv * g.y, x[i].z * inv * g.z, x[i].w * inv * g.w);
      if constexpr (CONV > 0) {
        // the input as it is kept, so that it counts the same now and as a past one
        Raw own;
        store4(reinterpret_cast<T*>(&own), y);
        const int taps = p.conv.taps;
        auto tap = [&](int j) { return *reinterpret_cast<const float4*>(p.conv.w + static_cast<size_t>(j) * H + c); };
        y = zero;
        if constexpr (CONV > 1) {
          const bool old = st != nullptr && !fresh;
#pragma unroll
          for (int j = 0; j < CONV - 1; ++j) {
            if (j >= taps - 1) break;
            if (old) y = fma4(tap(j), Quad<T>::value(past[i][j]), y);
            if (st != nullptr && j > 0) {
              if (old) *reinterpret_cast<Raw*>(st + static_cast<size_t>(j - 1) * H + c) = past[i][j];
              else store4(st + static_cast<size_t>(j - 1) * H + c, zero);
            }
          }
          if (st != nullptr && taps > 1) *reinterpret_cast<Raw*>(st + static_cast<size_t>(taps - 2) * H + c) = own;
        }
        y = fma4(tap(taps - 1), Quad<T>::value(own), y);
      }
      store4(p.out + ob + c, y);
    }
  } else {
    const int first = threadIdx.x, step = blockDim.x;
    if (p.conv.w != nullptr) st = conv_slot<T>(p.conv, row, H, fresh);
    float inv = 1.f;
    if (p.delta != nullptr && p.post != nullptr) {
      float ss = 0.f;
      for (int c = first; c < H; c += step) ss = fmaf(to_f(p.delta[in + c]), to_f(p.delta[in + c]), ss);
      inv = 1.f / sqrtf(block_sum(ss, red[0]) / H + p.eps);
    }
    float ss = 0.f;
    for (int c = first; c < H; c += step) {
      float x = p.residual[in + c];
      if (p.delta != nullptr) x = fmaf(to_f(p.delta[in + c]) * inv, p.post != nullptr ? to_f(p.post[c]) : 1.f, x);
      if (p.streams != nullptr) {
        float sum = 0.f;
        for (int j = 0; j < p.index; ++j) sum = fmaf(p.dw[j], p.streams[j * p.pitch + in + c], sum);
        if (p.keep) p.streams[p.index * p.pitch + in + c] = x;
        x = fmaf(p.dw[p.index], x, sum);
      }
      if (p.res_out != nullptr) p.res_out[ob + c] = x;
      held[c] = x;
      ss = fmaf(x, x, ss);
    }
    inv = p.gain / sqrtf(block_sum(ss, red[0]) / H + p.eps);
    for (int c = first; c < H; c += step) {
      float y = held[c] * inv * to_f(p.w[c]);
      if (p.conv.w != nullptr) {
        T h;
        put(&h, y);
        const int taps = p.conv.taps;
        y = p.conv.w[static_cast<size_t>(taps - 1) * H + c] * to_f(h);
        for (int j = 0; j < taps - 1; ++j) {
          const T v = st != nullptr && !fresh ? st[static_cast<size_t>(j) * H + c] : T(0.f);
          y = fmaf(p.conv.w[static_cast<size_t>(j) * H + c], to_f(v), y);
          if (st != nullptr && j > 0) st[static_cast<size_t>(j - 1) * H + c] = v;
        }
        if (st != nullptr && taps > 1) st[static_cast<size_t>(taps - 2) * H + c] = h;
      }
      put(p.out + ob + c, y);
    }
  }
}

// ------------------------------------------------------------------------------------------------
// x[T, H] -> out[T, H] convolved over time.  Q channels per thread (16 bytes), grid (channels, runs of R rows).  Rows that lie
// in one sequence with all their predecessors in the step are loaded together; others look up each input.
// ------------------------------------------------------------------------------------------------
template <typename T>
struct Piece {
  static constexpr int Q = 16 / sizeof(T);
  float v[Q];
};
template <typename T>
__device__ __forceinline__ void unpack(const uint4& u, float (&v)[16 / sizeof(T)]) {
  if constexpr (sizeof(T) == 4) {
    const float* f = reinterpret_cast<const float*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = f[i];
  } else {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(h[i]);
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  }
}
template <typename T>
__device__ __forceinline__ uint4 pack(const float (&v)[16 / sizeof(T)]) {
  uint4 u;
  if constexpr (sizeof(T) == 4) {
    u = make_uint4(__float_as_uint(v[0]), __float_as_uint(v[1]), __float_as_uint(v[2]), __float_as_uint(v[3]));
  } else {
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
  }
  return u;
}

template <typename T, int TAPS, int R>
__global__ void __launch_bounds__(128)
input_conv_kernel(const T* __restrict__ x, T* __restrict__ out, int T_, int H, const InputConv p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  constexpr int Q = Piece<T>::Q;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * Q, t0 = blockIdx.y * R, t1 = min(T_, t0 + R);
  if (c >= H) return;
  float w[TAPS][Q];
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
#pragma unroll
    for (int i = 0; i < Q; i += 4) {
      const float4 f = *reinterpret_cast<const float4*>(p.w + static_cast<size_t>(j) * H + c + i);
      w[j][i] = f.x; w[j][i + 1] = f.y; w[j][i + 2] = f.z; w[j][i + 3] = f.w;
    }
  int b = sequence_of(p.cu, p.B, t0), end = p.cu[b + 1];
  const uint4* src = reinterpret_cast<const uint4*>(x + c);
  uint4* dst = reinterpret_cast<uint4*>(out + c);
  const int pitch = H / Q;                                 // 16-byte pieces per row
  auto emit = [&](int t, const uint4 (&in)[TAPS]) {
    float a[Q];
#pragma unroll
    for (int i = 0; i < Q; ++i) a[i] = 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      float v[Q];
      unpack<T>(in[j], v);
#pragma unroll
      for (int i = 0; i < Q; ++i) a[i] = fmaf(w[j][i], v[i], a[i]);
    }
    dst[static_cast<size_t>(t) * pitch] = pack<T>(a);
  };
  if (t0 - p.cu[b] >= TAPS - 1 && t1 == t0 + R && t1 <= end) {
    uint4 in[R + TAPS - 1];
#pragma unroll
    for (int j = 0; j < R + TAPS - 1; ++j) in[j] = src[static_cast<size_t>(t0 - (TAPS - 1) + j) * pitch];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      uint4 own[TAPS];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) own[j] = in[r + j];
      emit(t0 + r, own);
    }
    return;
  }
  for (int t = t0; t < t1; ++t) {
    while (t >= end) end = p.cu[++b + 1];                  // sequences without tokens in this step are skipped
    const int begin = p.cu[b], local = t - begin, slot = p.slots[b];
    const bool past = p.kv_lens[b] - (end - begin) > 0 && slot >= 0 && slot < p.num_slots;
    uint4 in[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int back = TAPS - 1 - j;
      in[j] = make_uint4(0, 0, 0, 0);
      if (local >= back)
        in[j] = src[static_cast<size_t>(t - back) * pitch];
      else if (past)
        in[j] = reinterpret_cast<const uint4*>(static_cast<const T*>(p.state) + c)[(static_cast<size_t>(slot) * (TAPS - 1) + TAPS - 1 + local - back) * pitch];
    }
    emit(t, in);
  }
}

// the same for any width and number of taps, a thread per channel and row
template <typename T>
__global__ void __launch_bounds__(256)
input_conv_any_kernel(const T* __restrict__ x, T* __restrict__ out, int H, const InputConv p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int c = blockIdx.x * blockDim.x + threadIdx.x, t = blockIdx.y;
  if (c >= H) return;
  const int b = sequence_of(p.cu, p.B, t), begin = p.cu[b], local = t - begin, slot = p.slots[b];
  const bool past = p.kv_lens[b] - (p.cu[b + 1] - begin) > 0 && slot >= 0 && slot < p.num_slots;
  const T* st = static_cast<const T*>(p.state) + static_cast<size_t>(past ? slot : 0) * (p.taps - 1) * H + c;
  float a = 0.f;
  for (int j = 0; j < p.taps; ++j) {
    const int back = p.taps - 1 - j;
    float v = 0.f;
    if (local >= back) v = to_f(x[static_cast<size_t>(t - back) * H + c]);
    else if (past) v = to_f(st[static_cast<size_t>(p.taps - 1 + local - back) * H]);
    a = fmaf(p.w[static_cast<size_t>(j) * H + c], v, a);
  }
  put(out + static_cast<size_t>(t) * H + c, a);
}

// last taps - 1 inputs of every sequence that brought tokens -> its state.  Grid (channels, B)
template <typename T>
__global__ void __launch_bounds__(256)
input_conv_state_kernel(const T* __restrict__ x, int H, const InputConv p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int b = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int begin = p.cu[b], n = p.cu[b + 1] - begin, slot = p.slots[b];
  if (c >= H || n <= 0 || slot < 0 || slot >= p.num_slots) return;
  const bool fresh = p.kv_lens[b] - n <= 0;
  T* st = static_cast<T*>(p.state) + static_cast<size_t>(slot) * (p.taps - 1) * H + c;
  for (int j = 0; j < p.taps - 1; ++j) {                   // ascending: entry j is only read by entries before it
    const int i = n - (p.taps - 1) + j;                    // local index of the input that belongs at entry j
    T v = T(0.f);
    if (i >= 0) v = x[static_cast<size_t>(begin + i) * H + c];
    else if (!fresh) v = st[static_cast<size_t>(p.taps - 1 + i) * H];
    st[static_cast<size_t>(j) * H] = v;
  }
}

int done() { return cudaGetLastError() == cudaSuccess ? 0 : -3; }

template <typename T>
int stream_step(const StreamStep<T>& p, int n, cudaStream_t stream) {
  const int H = p.H, vecs = H / 4;
  if (H % 4 == 0 && vecs <= 2048 && (p.conv.w == nullptr || p.conv.taps <= kMaxTaps)) {
    const int most = p.conv.w != nullptr ? 1024 : 512, threads = vecs >= most ? most : ((vecs + 31) / 32) * 32;
    const int vpt = (vecs + threads - 1) / threads;
    auto go = [&](auto kern) {
      tgi::launch(kern, dim3(n), dim3(threads), 0, stream, p);
      return done();
    };
    auto pick = [&](auto avg) {
      constexpr bool A = decltype(avg)::value;
      if (p.conv.w == nullptr)
        return vpt <= 1 ? go(stream_step_kernel<T, 1, 0, A>) : vpt <= 2 ? go(stream_step_kernel<T, 2, 0, A>) : go(stream_step_kernel<T, 4, 0, A>);
      if (p.conv.taps <= 4) return vpt <= 1 ? go(stream_step_kernel<T, 1, 4, A>) : go(stream_step_kernel<T, 2, 4, A>);
      return vpt <= 1 ? go(stream_step_kernel<T, 1, kMaxTaps, A>) : go(stream_step_kernel<T, 2, kMaxTaps, A>);
    };
    return p.streams != nullptr ? pick(std::true_type()) : pick(std::false_type());
  }
  const size_t smem = static_cast<size_t>(H) * 4;
  if (smem > 200 * 1024) return -12;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(stream_step_kernel<T, 0, 1, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)
    return -2;
  tgi::launch(stream_step_kernel<T, 0, 1, true>, dim3(n), dim3(256), smem, stream, p);
  return done();
}

template <typename T>
int input_conv(const void* x, void* out, int T_, int H, const InputConv& p, cudaStream_t stream) {
  const T* src = static_cast<const T*>(x);
  constexpr int Q = Piece<T>::Q, R = 8;
  auto go = [&](auto kern) {
    const int pieces = H / Q, threads = pieces >= 128 ? 128 : (pieces + 31) / 32 * 32;
    tgi::launch(kern, dim3((pieces + threads - 1) / threads, (T_ + R - 1) / R), dim3(threads), 0, stream, src, static_cast<T*>(out),
                T_, H, p);
  };
  const bool vec = H % Q == 0 && (T_ + R - 1) / R <= 65535;
  if (vec && p.taps == 2) go(input_conv_kernel<T, 2, R>);
  else if (vec && p.taps == 3) go(input_conv_kernel<T, 3, R>);
  else if (vec && p.taps == 4) go(input_conv_kernel<T, 4, R>);
  else if (T_ <= 65535) tgi::launch(input_conv_any_kernel<T>, dim3((H + 255) / 256, T_), dim3(256), 0, stream, src, static_cast<T*>(out), H, p);
  else return -15;
  if (p.taps > 1) tgi::launch(input_conv_state_kernel<T>, dim3((H + 255) / 256, p.B), dim3(256), 0, stream, src, H, p);
  return done();
}

}  // namespace

// `f32` selects the build: 1 = fp32 activations and weights, 0 = bf16.
extern "C" {

// delta, post, rows, res_out may be null.  streams (optional): [index + 1 ..][..][H] with dw [index + 1]; keep: the new stream
// is stored there.  conv_w (optional): [taps][H], then every sequence brings at most one token.
int tgi_stream_step(int f32, const void* delta, const void* post, const float* residual, const int* rows, float* streams,
                    const float* dw, long long pitch, int index, int keep, const void* w, float gain, void* out, float* res_out,
                    int n, int H, float eps, const float* conv_w, const int* cu, const int* kv_lens, const int* slots, void* state,
                    int B, int taps, int num_slots, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (H < 1 || (streams != nullptr && (dw == nullptr || index < 0)) || (conv_w != nullptr && (taps < 1 || B < 1 || rows != nullptr)))
    return -10;
  const InputConv conv{conv_w, cu, kv_lens, slots, state, B, taps, num_slots};
  auto go = [&](auto tag) {
    using E = decltype(tag);
    const StreamStep<E> p{static_cast<const E*>(delta), static_cast<const E*>(post), static_cast<const E*>(w), residual, rows, streams,
                          dw, pitch, static_cast<E*>(out), res_out, H, index, keep, eps, gain, conv};
    return stream_step<E>(p, n, stream);
  };
  return f32 ? go(float()) : go(bf16());
}

// out may not be x; the sequences' states are advanced
int tgi_input_conv(int f32, const void* x, void* out, int T, int H, const float* w, const int* cu, const int* kv_lens,
                   const int* slots, void* state, int B, int taps, int num_slots, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (B < 1 || B > 65535 || taps < 1 || H < 1 || x == out) return -10;
  const InputConv p{w, cu, kv_lens, slots, state, B, taps, num_slots};
  return f32 ? input_conv<float>(x, out, T, H, p, stream) : input_conv<bf16>(x, out, T, H, p, stream);
}

}  // extern "C"
