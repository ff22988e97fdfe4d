// Paged causal attention over latents on the 5th-generation tensor cores (sm_100a), bf16.  Every token keeps one row that
// all query heads share: value columns first (the latent), then columns that only the keys have (a rotated part).  A row is
// read from memory once per tile of query rows; a query row is a (token, head) pair.
//
// A CTA owns N query rows (16, 32 or 64) and walks a range of keys in tiles of 128.  Both products are transposed, so that
// the 128 keys (or 128 value columns) are the rows of the MMA and a tile of few query rows wastes nothing:
//   S^T = K Q^T     M 128 (keys) x N x K width; the tile's slabs of 64 columns are multiplied as they land
//   P^T = softmax   four warps, a key per thread: column maxima by a transposing butterfly and shared memory, P^T as bf16
//                   rows [key][N] in shared memory (MN-major operand B)
//   O^T = V^T P^T   M 128 (value columns) x N x K 128 (keys), one product per 128 value columns; V^T is the K tile as it
//                   lies, taken as the MN-major operand A
// The output stays in registers of the output warps (a value column per thread, N query rows), which rescale it and add
// the tile's product.  The K tile is held once: a pair of slabs is loaded again as soon as its O^T product is done, the
// key-only slabs as soon as S^T is.  Pages (16 tokens) are fetched as TMA boxes of 16 rows x 128 bytes, the query rows as
// boxes of N rows.
//
// Decode steps (one token per sequence) run persistently: the key tiles of all sequences form one list that the CTAs
// share out evenly; a CTA's first and last piece may be parts of a sequence and go to a workspace that a second kernel
// merges.  Other steps run a CTA per tile of query rows.
// Every wait is bounded; a thread whose wait ran out sets the status word and does not wait again.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <atomic>

#include "launch.cuh"
#include "sm100.cuh"
#include "tensor_map.cuh"

using namespace sm100;

namespace {

constexpr int kKeys = 128, kPage = 16;
constexpr int kSlab = kKeys * 128;              // bytes of 64 columns of a K tile
constexpr int kMaxSlabs = 12, kMaxSeqs = 1024;
constexpr float kLog2e = 1.4426950408889634f;

struct LatentParams {
  const int *block_tables, *cu, *kv_lens;
  const __nv_bfloat16* gate;      // [T, ld_gate] or null: pre-activation of the factor on a head's output
  long long ld_gate;
  __nv_bfloat16* out;             // [T * H, out_cols]
  float *part_o, *part_ml;        // [2 * CTAs][N][out_cols] and [2 * CTAs][N][2]
  int* range;                     // [items][2]: first and last CTA of an item (persistent)
  int B, max_blocks, num_blocks, H, out_cols, slabs, value_slabs, window, persistent, most;
  float scale_log2;
  int* status;
};

__device__ __forceinline__ void report(int* status, int code) {
  if (status != nullptr) atomicCAS(status, 0, code);
}
__device__ __forceinline__ uint64_t desc_mn(uint32_t addr, uint32_t lbo) {      // MN-major, 128-byte swizzle
  uint64_t d = 0;
  d |= static_cast<uint64_t>((addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>(lbo >> 4) << 16;
  d |= static_cast<uint64_t>(1024 >> 4) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <int W>
__device__ __forceinline__ void tmem_load(uint32_t addr, float (&v)[W]) {
  static_assert(W == 16 || W == 32, "columns of one load");
  uint32_t r[W];
  if constexpr (W == 32) {
    tmem_ld_32x32b_x32(addr, r);
    tmem_ld_wait(r);
  } else {
    tmem_ld_32x32b_x16(addr, r);
    asm volatile("tcgen05.wait::ld.sync.aligned;"
                 : "+r"(r[0]), "+r"(r[1]), "+r"(r[2]), "+r"(r[3]), "+r"(r[4]), "+r"(r[5]), "+r"(r[6]), "+r"(r[7]),
                   "+r"(r[8]), "+r"(r[9]), "+r"(r[10]), "+r"(r[11]), "+r"(r[12]), "+r"(r[13]), "+r"(r[14]), "+r"(r[15])
                 :
                 : "memory");
  }
#pragma unroll
  for (int i = 0; i < W; ++i) v[i] = __uint_as_float(r[i]);
}
// W values per lane -> lane l gets the maximum (sum) of value l % W over the warp
template <int W, bool SUM>
__device__ __forceinline__ float column_reduce(float (&v)[W], int lane) {
#pragma unroll
  for (int o = W / 2; o >= 1; o >>= 1) {
    const bool up = (lane & o) != 0;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float keep = up ? v[i + o] : v[i], send = up ? v[i] : v[i + o];
      const float got = __shfl_xor_sync(0xffffffffu, send, o);
      v[i] = SUM ? keep + got : fmaxf(keep, got);
    }
  }
#pragma unroll
  for (int o = W; o < 32; o <<= 1) {
    const float got = __shfl_xor_sync(0xffffffffu, v[0], o);
    v[0] = SUM ? v[0] + got : fmaxf(v[0], got);
  }
  return v[0];
}
__device__ __forceinline__ int first_visible(int pos, int window) { return window > 0 ? max(0, pos - window + 1) : 0; }
// key tiles of the rows whose first and last token sit at pos0 and pos1 (at least one: its keys are masked), and their start
__device__ __forceinline__ int tiles_of(int pos0, int pos1, int window, int& t_lo) {
  t_lo = first_visible(pos0, window) / kPage * kPage;
  return max(1, (pos1 + 1 - t_lo + kKeys - 1) / kKeys);
}

// ---- work list -------------------------------------------------------------------------------------
struct Piece {
  int b, row0, rows, q_row;       // query rows [row0, row0 + N) of the sequence, of which `rows` exist; q_row: first in [T * H]
  int pos0, pos1;                 // positions of the first and the last row's token
  int t_lo, first, tiles;         // first key of the item, first tile and number of tiles of this piece
  int part;                       // -1: the whole item, else which of the CTA's workspace slots
  int item, last_cta;             // persistent: number of the item, CTA that ends it
};
// tiles before sequence b of a decode step (one warp; every item of a sequence has the same number of tiles)
__device__ __forceinline__ void decode_prefix(const LatentParams& p, int* prefix, int lane) {
  int sum = 0;
  for (int b0 = 0; b0 < p.B; b0 += 32) {
    const int b = b0 + lane;
    int v = 0, t_lo;
    if (b < p.B && p.cu[b + 1] > p.cu[b]) v = tiles_of(p.kv_lens[b] - 1, p.kv_lens[b] - 1, p.window, t_lo);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int got = __shfl_up_sync(0xffffffffu, v, o);
      if (lane >= o) v += got;
    }
    if (b < p.B) prefix[b + 1] = sum + v;
    sum += __shfl_sync(0xffffffffu, v, 31);
  }
  if (lane == 0) prefix[0] = 0;
}
__device__ __forceinline__ int sequence_at(const int* prefix, int B, int items, long long g) {
  int lo = 0, hi = B - 1;         // the last b with prefix[b] * items <= g that has tiles
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (static_cast<long long>(prefix[mid]) * items <= g) lo = mid;
    else hi = mid - 1;
  }
  return lo;
}
template <int N>
struct Walk {
  long long g, end, total;        // persistent: tiles of the list that are left, and all
  int items;
  __device__ __forceinline__ void start(const LatentParams& p, const int* prefix) {
    items = (p.H + N - 1) / N;
    g = 0;
    end = 1;
    if (p.persistent) {
      total = static_cast<long long>(prefix[p.B]) * items;
      g = total * blockIdx.x / gridDim.x;
      end = total * (blockIdx.x + 1) / gridDim.x;
    }
  }
  __device__ __forceinline__ bool next(const LatentParams& p, const int* prefix, Piece& w) {
    if (g >= end) return false;
    int rt;
    if (p.persistent) {
      w.b = sequence_at(prefix, p.B, items, g);
      const int nt = prefix[w.b + 1] - prefix[w.b];
      const long long at = g - static_cast<long long>(prefix[w.b]) * items;
      rt = static_cast<int>(at / nt);
      w.first = static_cast<int>(at - static_cast<long long>(rt) * nt);
      w.tiles = static_cast<int>(min(static_cast<long long>(nt - w.first), end - g));
      w.part = w.first == 0 && w.tiles == nt ? -1 : (w.first == 0 ? 1 : 0);
      w.item = w.b * items + rt;
      w.last_cta = static_cast<int>(((g - w.first + nt) * gridDim.x - 1) / total);
      g += w.tiles;
    } else {
      w.b = blockIdx.y;
      rt = gridDim.x - 1 - blockIdx.x;                     // long items first
      w.first = 0;
      w.part = -1;
      g = end;
    }
    const int begin = p.cu[w.b], n = p.cu[w.b + 1] - begin;
    w.row0 = rt * N;
    w.rows = min(N, n * p.H - w.row0);
    if (w.rows <= 0 || n > p.most) return false;           // not persistent: nothing here
    w.q_row = begin * p.H + w.row0;
    const int base = p.kv_lens[w.b] - n;
    w.pos0 = base + w.row0 / p.H;
    w.pos1 = base + (w.row0 + w.rows - 1) / p.H;
    const int nt = tiles_of(w.pos0, w.pos1, p.window, w.t_lo);
    if (!p.persistent) w.tiles = nt;
    return true;
  }
};

// bounded wait that a thread gives up on once
struct Waiter {
  int* status;
  bool failed;
  __device__ __forceinline__ bool operator()(uint64_t* bar, uint32_t parity, int code) {
    if (!failed && !mbar_wait(bar, parity)) {
      report(status, code);
      failed = true;
    }
    return !failed;
  }
};

template <int N, int OG>
__global__ void __launch_bounds__(256 + 128 * OG, 1)
latent_attention_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const LatentParams p) {
  constexpr int W = N < 32 ? N : 32;            // columns per TMEM load
  constexpr int NB = N == 64 ? 1 : 2;           // blocks of 128 value columns per output warp group
  extern __shared__ __align__(1024) uint8_t smem[];
  if ((smem_u32(smem) & 1023u) != 0u) {         // uniform over the CTA, before anything is allocated
    if (threadIdx.x == 0) report(p.status, kErrSmemLayout);
    return;
  }
  const int blocks = (p.value_slabs + 1) / 2, held = max(p.slabs, 2 * blocks);
  uint8_t* sK = smem;
  uint8_t* sQ = sK + held * kSlab;              // [slab][N rows of 128 bytes]
  uint8_t* sP = sQ + p.slabs * N * 128;         // [key][64 columns]
  float* s_max = reinterpret_cast<float*>(sP + kKeys * 128);      // [4][N] maxima of the softmax warps
  float* s_m = s_max + 4 * N;                   // [N]
  float* s_alpha = s_m + N;                     // [N]
  float* s_l = s_alpha + N;                     // [N] factor of the output
  int* s_lo = reinterpret_cast<int*>(s_l + N);  // [N] first and last visible key of a row
  int* s_hi = s_lo + N;
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_hi + N);
  uint64_t* k_full = bars;                      // [kMaxSlabs]
  uint64_t* k_free = bars + kMaxSlabs;          // [kMaxSlabs / 2] by the O^T product of a block
  uint64_t* kk_free = k_free + kMaxSlabs / 2;   // key-only slabs, by S^T
  uint64_t* q_full = kk_free + 1;
  uint64_t* q_free = q_full + 1;
  uint64_t* s_full = q_full + 2;
  uint64_t* p_ready = q_full + 3;
  uint64_t* o_full = q_full + 4;
  uint64_t* o_free = q_full + 5;
  uint64_t* l_ready = q_full + 6;
  uint64_t* l_free = q_full + 7;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(q_full + 8);
  int* prefix = reinterpret_cast<int*>(tmem_holder + 4);          // [B + 1], persistent only

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  uint32_t cols = 32;
  while (static_cast<int>(cols) < N * (1 + blocks)) cols <<= 1;
  if (threadIdx.x == 0) {
    for (int i = 0; i < kMaxSlabs; ++i) mbar_init(&k_full[i], 1);
    for (int i = 0; i < kMaxSlabs / 2; ++i) mbar_init(&k_free[i], 1);
    mbar_init(kk_free, 1);
    mbar_init(q_full, 1);
    mbar_init(q_free, 1);
    mbar_init(s_full, 1);
    mbar_init(p_ready, 4);
    mbar_init(o_full, 1);
    mbar_init(o_free, 4 * OG);
    mbar_init(l_ready, 4);
    mbar_init(l_free, 4 * OG);
    fence_barrier_init();
    prefetch_tensormap(&tmQ);
    prefetch_tensormap(&tmK);
  }
  if (warp == 1) {
    tmem_alloc(tmem_holder, cols);
    tmem_relinquish();
  }
  tgi::pdl_wait();
  tgi::pdl_trigger();
  if (warp == 2 && p.persistent) decode_prefix(p, prefix, lane);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tS = *tmem_holder, tO = tS + N;
  Waiter wait{p.status, false};
  Walk<N> walk;
  walk.start(p, prefix);
  Piece w;
  int j = 0, np = 0;                            // tiles and pieces so far

  if (warp == 0) {
    // ---------------- TMA producer: a box of 16 rows x 128 bytes per page and slab, spread over the lanes ----------------
    bool ok = true;
    auto slab_pair = [&](int s0, int count, int blk, bool go) {     // slabs s0 .. s0 + count - 1 (at most two)
      if (lane == 0 && go)
        for (int i = 0; i < count; ++i) mbar_arrive_expect_tx(&k_full[s0 + i], kSlab);
      __syncwarp();
      const int s = s0 + (lane >> 3), pg = lane & 7;
      if (go && (lane >> 3) < count)
        tma_load_2d(sK + s * kSlab + pg * (kPage * 128), &tmK, &k_full[s], s * 64, blk * kPage);
    };
    while (ok && walk.next(p, prefix, w)) {
      if (np > 0) ok = wait(q_free, (np - 1) & 1, kErrProducerWait);
      ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
      if (!ok) break;
      if (lane == 0) mbar_arrive_expect_tx(q_full, p.slabs * N * 128);
      __syncwarp();
      if (lane < p.slabs) tma_load_2d(sQ + lane * N * 128, &tmQ, q_full, lane * 64, w.q_row);
      for (int i = 0; i < w.tiles && ok; ++i, ++j) {
        const int page = (w.t_lo + (w.first + i) * kKeys) / kPage + (lane & 7);
        int blk = 0;
        if (page < p.max_blocks) blk = p.block_tables[static_cast<size_t>(w.b) * p.max_blocks + page];
        blk = min(max(blk, 0), p.num_blocks - 1);          // pages past the sequence are masked later
        for (int s = p.value_slabs; s < p.slabs && ok; s += 2) {
          if (s == p.value_slabs && j > 0) ok = wait(kk_free, (j - 1) & 1, kErrProducerWait);
          ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
          slab_pair(s, min(2, p.slabs - s), blk, ok);
        }
        for (int b = 0; b < blocks && ok; ++b) {
          if (j > 0) ok = wait(&k_free[b], (j - 1) & 1, kErrProducerWait);
          ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
          slab_pair(2 * b, min(2, p.value_slabs - 2 * b), blk, ok);
        }
      }
      ++np;
    }
    // copies in flight must land before the CTA's shared memory goes away (after a failed wait: also those of the
    // tile that was being requested, as far as they were)
    if (lane == 0) {
      for (int s = 0; s < p.slabs; ++s) {
        if (j > 0) mbar_wait(&k_full[s], (j - 1) & 1);
        if (!ok) mbar_wait(&k_full[s], j & 1);
      }
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (elect_one()) {
      constexpr uint32_t id_s = (1u << 4) | (1u << 7) | (1u << 10) | ((static_cast<uint32_t>(N) >> 3) << 17) | ((128u >> 4) << 24);
      constexpr uint32_t id_o = id_s | (1u << 15) | (1u << 16);          // both operands MN-major
      const uint32_t q_addr = smem_u32(sQ), k_addr = smem_u32(sK), p_addr = smem_u32(sP);
      bool ok = true;
      while (ok && walk.next(p, prefix, w)) {
        ok = wait(q_full, np & 1, kErrMmaWaitFull);
        for (int i = 0; i < w.tiles && ok; ++i, ++j) {
          // S^T: key-only slabs first, they land first
          for (int x = 0; x < p.slabs && ok; ++x) {
            const int s = x < p.slabs - p.value_slabs ? p.value_slabs + x : x - (p.slabs - p.value_slabs);
            ok = wait(&k_full[s], j & 1, kErrMmaWaitFull);
            if (!ok) break;
            tc_fence_after();
#pragma unroll
            for (int k = 0; k < 4; ++k)
              mma_f16(tS, make_desc_sw128(k_addr + s * kSlab) + (k * 32 >> 4), make_desc_sw128(q_addr + s * N * 128) + (k * 32 >> 4), id_s,
                      x > 0 || k > 0 ? 1u : 0u);
          }
          if (!ok) break;
          tc_commit(s_full);
          tc_commit(kk_free);
          if (i + 1 == w.tiles) tc_commit(q_free);
          ok = wait(p_ready, j & 1, kErrMmaWaitFull);
          if (!ok) break;
          tc_fence_after();
          for (int b = 0; b < blocks; ++b) {
#pragma unroll
            for (int k = 0; k < 8; ++k)                    // 16 keys: two groups of eight 128-byte rows
              mma_f16(tO + b * N, desc_mn(k_addr + 2 * b * kSlab + k * 2048, kSlab), desc_mn(p_addr + k * 2048, kSlab), id_o,
                      k > 0 ? 1u : 0u);
            tc_commit(&k_free[b]);
          }
          tc_commit(o_full);
        }
        ++np;
      }
    }
  } else if (warp >= 4 && warp < 8) {
    // ---------------- softmax: a key per thread ----------------
    const int quarter = warp & 3, key = quarter * 32 + lane;
    const uint32_t addr = tS + (static_cast<uint32_t>(quarter * 32) << 16);
    while (walk.next(p, prefix, w)) {
      const int t_end = w.t_lo + w.first * kKeys;          // first key of the piece
      float l[N];
#pragma unroll
      for (int c = 0; c < N; ++c) l[c] = 0.f;
      float m = -INFINITY;                                 // thread c < N: running maximum of row c
      if (key < N) {
        const int pos = w.pos0 + (w.row0 % p.H + min(key, w.rows - 1)) / p.H;
        s_lo[key] = first_visible(pos, p.window);
        s_hi[key] = pos;
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      // keys that every row sees
      const int lo_all = first_visible(w.pos1, p.window), hi_all = w.pos0;
      for (int i = 0; i < w.tiles; ++i, ++j) {
        const int t0 = t_end + i * kKeys, t = t0 + key;
        const bool plain = t0 >= lo_all && t0 + kKeys - 1 <= hi_all;
        auto score = [&](float x, int c) {
          return plain || (t >= s_lo[c] && t <= s_hi[c]) ? x * p.scale_log2 : -INFINITY;
        };
        wait(s_full, j & 1, kErrEpilogueWait);
        tc_fence_after();
#pragma unroll
        for (int c0 = 0; c0 < N; c0 += W) {
          float v[W];
          tmem_load<W>(addr + c0, v);
#pragma unroll
          for (int c = 0; c < W; ++c) v[c] = score(v[c], c0 + c);
          const float mx = column_reduce<W, false>(v, lane);
          if (lane < W) s_max[quarter * N + c0 + lane] = mx;
        }
        // the last tile's output has been taken: its factors and its P^T are free
        if (j > 0) wait(o_free, (j - 1) & 1, kErrEpilogueWait);
        asm volatile("bar.sync 1, 128;" ::: "memory");
        if (key < N) {
          const float mn = fmaxf(fmaxf(fmaxf(s_max[key], s_max[N + key]), fmaxf(s_max[2 * N + key], s_max[3 * N + key])), m);
          s_alpha[key] = mn == -INFINITY ? 1.f : ex2(m - mn);
          s_m[key] = mn == -INFINITY ? 0.f : mn;
          m = mn;
        }
        asm volatile("bar.sync 1, 128;" ::: "memory");
#pragma unroll
        for (int c0 = 0; c0 < N; c0 += W) {
          float v[W];
          tmem_load<W>(addr + c0, v);
#pragma unroll
          for (int c = 0; c < W; c += 8) {
            uint32_t packed[4];
#pragma unroll
            for (int e = 0; e < 8; e += 4) {
              const float4 mm = *reinterpret_cast<const float4*>(s_m + c0 + c + e);
              const float4 al = *reinterpret_cast<const float4*>(s_alpha + c0 + c + e);
              const float pr[4] = {ex2(score(v[c + e], c0 + c + e) - mm.x), ex2(score(v[c + e + 1], c0 + c + e + 1) - mm.y),
                                   ex2(score(v[c + e + 2], c0 + c + e + 2) - mm.z), ex2(score(v[c + e + 3], c0 + c + e + 3) - mm.w)};
              l[c0 + c + e] = fmaf(l[c0 + c + e], al.x, pr[0]);
              l[c0 + c + e + 1] = fmaf(l[c0 + c + e + 1], al.y, pr[1]);
              l[c0 + c + e + 2] = fmaf(l[c0 + c + e + 2], al.z, pr[2]);
              l[c0 + c + e + 3] = fmaf(l[c0 + c + e + 3], al.w, pr[3]);
              const __nv_bfloat162 a = __floats2bfloat162_rn(pr[0], pr[1]), b = __floats2bfloat162_rn(pr[2], pr[3]);
              packed[e / 2] = *reinterpret_cast<const uint32_t*>(&a);
              packed[e / 2 + 1] = *reinterpret_cast<const uint32_t*>(&b);
            }
            *reinterpret_cast<uint4*>(sP + key * 128 + ((((c0 + c) >> 3) ^ (key & 7)) << 4)) =
                make_uint4(packed[0], packed[1], packed[2], packed[3]);
          }
        }
        fence_proxy_async();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(p_ready);
      }
      // sums over the keys; what the output is multiplied by
#pragma unroll
      for (int c0 = 0; c0 < N; c0 += W) {
        float v[W];
#pragma unroll
        for (int c = 0; c < W; ++c) v[c] = l[c0 + c];
        const float sum = column_reduce<W, true>(v, lane);
        if (lane < W) s_max[quarter * N + c0 + lane] = sum;
      }
      if (np > 0) wait(l_free, (np - 1) & 1, kErrEpilogueWait);
      asm volatile("bar.sync 1, 128;" ::: "memory");
      if (key < N) {
        const float sum = (s_max[key] + s_max[N + key]) + (s_max[2 * N + key] + s_max[3 * N + key]);
        float f = 1.f;
        if (w.part < 0) {
          if (p.persistent && key == 0) p.range[2 * w.item] = p.range[2 * w.item + 1] = 0;
          f = sum > 0.f ? 1.f / sum : 0.f;
          if (p.gate != nullptr && key < w.rows) {
            const int row = w.q_row + key;
            f *= __fdividef(1.f, 1.f + __expf(-__bfloat162float(p.gate[static_cast<long long>(row / p.H) * p.ld_gate + row % p.H])));
          }
        } else {
          if (key == 0 && w.first == 0) {
            p.range[2 * w.item] = blockIdx.x;
            p.range[2 * w.item + 1] = w.last_cta;
          }
          float* ml = p.part_ml + (static_cast<size_t>(2 * blockIdx.x + w.part) * N + key) * 2;
          ml[0] = m;
          ml[1] = sum;
        }
        s_l[key] = f;
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(l_ready);
      ++np;
    }
  } else if (warp >= 8) {
    // ---------------- output: a value column per thread ----------------
    const int quarter = warp & 3, group = (warp - 8) >> 2;
    const uint32_t addr = tO + (static_cast<uint32_t>(quarter * 32) << 16);
    while (walk.next(p, prefix, w)) {
      float o[NB][N];
#pragma unroll
      for (int x = 0; x < NB; ++x)
#pragma unroll
        for (int c = 0; c < N; ++c) o[x][c] = 0.f;
      for (int i = 0; i < w.tiles; ++i, ++j) {
        wait(o_full, j & 1, kErrEpilogueWait);
        tc_fence_after();
#pragma unroll
        for (int x = 0; x < NB; ++x) {
          const int b = group + OG * x;
          if (b >= blocks) break;                          // warp-uniform
#pragma unroll
          for (int c0 = 0; c0 < N; c0 += W) {
            float v[W];
            tmem_load<W>(addr + b * N + c0, v);
#pragma unroll
            for (int c = 0; c < W; c += 4) {
              const float4 al = *reinterpret_cast<const float4*>(s_alpha + c0 + c);
              o[x][c0 + c] = fmaf(o[x][c0 + c], al.x, v[c]);
              o[x][c0 + c + 1] = fmaf(o[x][c0 + c + 1], al.y, v[c + 1]);
              o[x][c0 + c + 2] = fmaf(o[x][c0 + c + 2], al.z, v[c + 2]);
              o[x][c0 + c + 3] = fmaf(o[x][c0 + c + 3], al.w, v[c + 3]);
            }
          }
        }
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(o_free);
      }
      wait(l_ready, np & 1, kErrEpilogueWait);
      float* part = p.part_o + static_cast<size_t>(2 * blockIdx.x + max(w.part, 0)) * N * p.out_cols;
#pragma unroll
      for (int x = 0; x < NB; ++x) {
        const int col = (group + OG * x) * 128 + quarter * 32 + lane;
        if (col >= p.out_cols) continue;
#pragma unroll
        for (int c = 0; c < N; ++c) {
          if (c >= w.rows) break;
          if (w.part < 0) p.out[static_cast<size_t>(w.q_row + c) * p.out_cols + col] = __float2bfloat16(o[x][c] * s_l[c]);
          else part[static_cast<size_t>(c) * p.out_cols + col] = o[x][c];
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(l_free);
      ++np;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tS, cols);
}

// Items of a persistent launch that several CTAs shared.  Grid (items, groups of four query rows).
template <int N>
__global__ void __launch_bounds__(256)
latent_merge_kernel(const LatentParams p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  const int items = (p.H + N - 1) / N, b = blockIdx.x / items, rt = blockIdx.x % items;
  const int begin = p.cu[b], rows = min(N, p.H - rt * N);
  if (p.cu[b + 1] <= begin) return;
  const int c0 = p.range[2 * blockIdx.x], c1 = p.range[2 * blockIdx.x + 1];
  if (c0 == c1) return;                                    // one CTA did the whole item
  for (int i = threadIdx.x; i < 4 * p.out_cols; i += blockDim.x) {
    const int r = blockIdx.y * 4 + i / p.out_cols, col = i % p.out_cols;
    if (r >= rows) break;
    // the first of the CTAs ended with its part (slot 1), the others began with theirs (slot 0)
    auto slot = [&](int c) { return static_cast<size_t>(2 * c + (c == c0 ? 1 : 0)) * N + r; };
    float mm = -INFINITY, sum = 0.f, o = 0.f;
    for (int c = c0; c <= c1; ++c) mm = fmaxf(mm, p.part_ml[slot(c) * 2]);
    for (int c = c0; c <= c1; ++c) {
      const float m = p.part_ml[slot(c) * 2];
      if (m == -INFINITY) continue;
      const float f = exp2f(m - mm);
      sum = fmaf(p.part_ml[slot(c) * 2 + 1], f, sum);
      o = fmaf(p.part_o[slot(c) * p.out_cols + col], f, o);
    }
    float f = sum > 0.f ? 1.f / sum : 0.f;
    if (p.gate != nullptr)
      f *= __fdividef(1.f, 1.f + __expf(-__bfloat162float(p.gate[static_cast<long long>(begin) * p.ld_gate + rt * N + r])));
    p.out[(static_cast<size_t>(begin) * p.H + rt * N + r) * p.out_cols + col] = __float2bfloat16(o * f);
  }
}

int smem_bytes(int N, int slabs, int value_slabs, int seqs) {
  const int held = max(slabs, (value_slabs + 1) / 2 * 2);
  return held * kSlab + slabs * N * 128 + kKeys * 128 + 9 * N * 4 + (kMaxSlabs + kMaxSlabs / 2 + 9) * 8 + 16 + (seqs + 1) * 4;
}

template <int N, int OG>
int launch(const LatentParams& p, const void* q, const void* pages, long long q_rows, int max_q, int ctas, cudaStream_t stream) {
  CUtensorMap tmQ, tmK;
  const uint64_t width = static_cast<uint64_t>(p.slabs) * 64;
  int rc = tgi::make_map_2d(&tmQ, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, q, q_rows, width, width * 2, N, 64, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  rc = tgi::make_map_2d(&tmK, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, pages, static_cast<uint64_t>(p.num_blocks) * kPage, width, width * 2,
                        kPage, 64, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  auto kern = latent_attention_kernel<N, OG>;
  static std::atomic<unsigned long long> attr_set{0};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess) return -2;
  const unsigned long long bit = 1ull << (dev & 63);
  if (!(attr_set.load(std::memory_order_acquire) & bit)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -2;
    attr_set.fetch_or(bit, std::memory_order_release);
  }
  const int items = (max_q * p.H + N - 1) / N;
  const dim3 grid = p.persistent ? dim3(ctas) : dim3(items, p.B);
  const size_t smem = smem_bytes(N, p.slabs, p.value_slabs, p.persistent ? p.B : 0);
  tgi::launch(kern, grid, dim3(256 + 128 * OG), smem, stream, tmQ, tmK, p);
  if (p.persistent) tgi::launch(latent_merge_kernel<N>, dim3(p.B * items, (min(N, p.H) + 3) / 4), dim3(256), 0, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace

extern "C" {

// Query rows per tile for rows of `slabs` x 64 columns, `value_slabs` of them values; 0: the kernel does not take them.
int tgi_latent_rows(int slabs, int value_slabs, long long rows) {
  if (value_slabs < 1 || value_slabs > 8 || slabs < value_slabs || slabs > kMaxSlabs) return 0;
  int N = rows <= 16 ? 16 : rows <= 32 || value_slabs > 4 ? 32 : 64;
  while (N >= 16 && smem_bytes(N, slabs, value_slabs, kMaxSeqs) > 227 * 1024) N /= 2;
  return N >= 16 ? N : 0;
}

// q [T, H, slabs * 64] and pages [num_blocks, 16, slabs * 64] bf16 (the first value_slabs * 64 columns of a row are the
// values), out [T, H, value_slabs * 64].  part_o / part_ml: 2 * ctas slots of N x (value_slabs * 64) and N x 2 floats, range:
// 2 * B * ceil(H / N) ints; used when max_q == 1.  Sequences with more than `most` tokens are left out.  gate (optional): [T, ld_gate].
int tgi_latent_attention(const void* q, const void* pages, const int* block_tables, const int* cu, const int* kv_lens,
                         const void* gate, long long ld_gate, void* out, float* part_o, float* part_ml, int* range, int T, int B, int max_q,
                         int max_blocks, int num_blocks, int H, int slabs, int value_slabs, int N, float scale, int window,
                         int most, int ctas, int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || max_q <= 0) return 0;
  if (N != 16 && N != 32 && N != 64) return -10;
  if (B > 65535 || num_blocks < 1 || max_blocks < 1 || ctas < 1 || smem_bytes(N, slabs, value_slabs, kMaxSeqs) > 227 * 1024) return -10;
  LatentParams p;
  p.block_tables = block_tables;
  p.cu = cu;
  p.kv_lens = kv_lens;
  p.gate = static_cast<const __nv_bfloat16*>(gate);
  p.ld_gate = ld_gate;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.part_o = part_o;
  p.part_ml = part_ml;
  p.range = range;
  p.B = B;
  p.max_blocks = max_blocks;
  p.num_blocks = num_blocks;
  p.H = H;
  p.out_cols = value_slabs * 64;
  p.slabs = slabs;
  p.value_slabs = value_slabs;
  p.window = window;
  p.persistent = max_q == 1 && B <= kMaxSeqs && part_o != nullptr && part_ml != nullptr && range != nullptr;
  p.most = most;
  p.scale_log2 = scale * kLog2e;
  p.status = status;
  const long long rows = static_cast<long long>(T) * H;
  const bool wide = value_slabs > 4;
  if (N == 64) return wide ? -10 : launch<64, 2>(p, q, pages, rows, max_q, ctas, stream);
  if (N == 32) return wide ? launch<32, 2>(p, q, pages, rows, max_q, ctas, stream) : launch<32, 1>(p, q, pages, rows, max_q, ctas, stream);
  return wide ? launch<16, 2>(p, q, pages, rows, max_q, ctas, stream) : launch<16, 1>(p, q, pages, rows, max_q, ctas, stream);
}

}  // extern "C"
