// Paged causal attention over latents on the 5th-generation tensor cores (sm_100a), bf16.  Every token keeps one row that
// all query heads share: value columns first (the latent), then columns that only the keys have (a rotated part).  A row is
// read from memory once per tile of query rows; a query row is a (token, head) pair.
//
// A CTA owns N query rows (16, 32 or 64) and walks a range of keys in tiles of 64.  Both products are transposed, so that
// keys (or value columns) are the rows of the MMA and a tile of few query rows wastes nothing:
//   S^T = K Q^T     M 64 (keys) x N x K width
//   P^T = softmax   four warps, half of the query rows of a key per thread, P^T as bf16 rows [key][N] in shared memory
//                   (MN-major operand B).  The maximum that the exponents refer to is kept while no score passes it by
//                   more than kSlack (one reducing barrier tells); otherwise column maxima are taken by a transposing
//                   butterfly and shared memory, and sums and outputs are rescaled
//   O^T = V^T P^T   M 128 (value columns) x N x K 64 (keys), one product per 128 value columns; V^T is the K tile as it
//                   lies, taken as the MN-major operand A
// The output stays in registers of the output warps (a value column per thread, N query rows), which rescale it and add
// the tile's product.  S^T, P^T and O^T are double-buffered and S^T of a tile is issued before O^T of the tile in front of
// it when the tile has landed by then.
//
// A page (16 tokens) is one TMA box: [8 tokens x 128 bytes] atoms of the 128-byte swizzle, first along the row, then the
// other 8 tokens.  Groups of 8 keys are thus `slabs` KB apart in shared memory, which both operand descriptors take as a
// stride; a copy of 2 KB boxes (page x 128 bytes) ran at half the rate, a thread's copies issue one after the other.
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

constexpr int kKeys = 64, kPage = 16;
constexpr int kMaxSlabs = 12, kMaxSeqs = 1024, kMaxStages = 4;
constexpr int kPTile = kKeys * 128;             // bytes of a P^T tile
constexpr float kSlack = 8.f;                   // log2: probabilities stay below 256 times those of the true maximum
constexpr float kNoMax = -1e30f;                // maximum of no key
constexpr float kLog2e = 1.4426950408889634f;

struct LatentParams {
  const int *block_tables, *cu, *kv_lens;
  const int* elsewhere;           // null, or [B]: sequences whose entry is at least their number of tokens are left out
  const __nv_bfloat16* gate;      // [T, ld_gate] or null: pre-activation of the factor on a head's output
  long long ld_gate;
  const float* sink;              // [H] or null: score of one more key per head that has no value
  __nv_bfloat16* out;             // [T * H, out_cols]
  float *part_o, *part_ml;        // [2 * CTAs][N][out_cols] and [2 * CTAs][N][2]
  int* range;                     // [items][2]: first and last CTA of an item (persistent)
  int B, max_blocks, num_blocks, H, out_cols, slabs, value_slabs, stages, window, persistent;
  float scale_log2;
  int* status;
};

__device__ __forceinline__ void report(int* status, int code) {
  if (status != nullptr) atomicCAS(status, 0, code);
}
// 128-byte swizzle.  K-major: groups of 8 rows `sbo` bytes apart.  MN-major: groups of 8 K rows `sbo` bytes apart, the next
// 64 elements of M or N `lbo` bytes further.
__device__ __forceinline__ uint64_t make_desc(uint32_t addr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>(lbo >> 4) << 16;
  d |= static_cast<uint64_t>(sbo >> 4) << 32;
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
// C values per lane -> lane l gets the maximum (sum) of value l % C over the 16 lanes of its half warp
template <int C, bool SUM>
__device__ __forceinline__ float column_reduce(float (&v)[C], int lane) {
#pragma unroll
  for (int o = C / 2; o >= 1; o >>= 1) {
    const bool up = (lane & o) != 0;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float keep = up ? v[i + o] : v[i], send = up ? v[i] : v[i + o];
      const float got = __shfl_xor_sync(0xffffffffu, send, o);
      v[i] = SUM ? keep + got : fmaxf(keep, got);
    }
  }
#pragma unroll
  for (int o = C; o < 16; o <<= 1) {
    const float got = __shfl_xor_sync(0xffffffffu, v[0], o);
    v[0] = SUM ? v[0] + got : fmaxf(v[0], got);
  }
  return v[0];
}
// the sink's share of the denominator of head h, for exponents that refer to m
__device__ __forceinline__ float sink_term(const float* sink, int h, float m) {
  return sink != nullptr ? exp2f(fmaf(sink[h], kLog2e, -m)) : 0.f;
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
__device__ __forceinline__ bool taken(const LatentParams& p, int b) {
  const int n = p.cu[b + 1] - p.cu[b];
  return n > 0 && (p.elsewhere == nullptr || p.elsewhere[b] < n);
}
// Tiles before sequence b of a decode step (every item of a sequence has the same number of tiles): the whole CTA looks up
// the sequences, one warp adds up.
__device__ __forceinline__ void decode_tiles(const LatentParams& p, int* prefix) {
  for (int b = threadIdx.x; b < p.B; b += blockDim.x) {
    int t_lo;
    prefix[b + 1] = taken(p, b) ? tiles_of(p.kv_lens[b] - 1, p.kv_lens[b] - 1, p.window, t_lo) : 0;
  }
  if (threadIdx.x == 0) prefix[0] = 0;
}
__device__ __forceinline__ void decode_prefix(const LatentParams& p, int* prefix, int lane) {
  int sum = 0;
  for (int b0 = 0; b0 < p.B; b0 += 32) {
    const int b = b0 + lane;
    int v = b < p.B ? prefix[b + 1] : 0;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int got = __shfl_up_sync(0xffffffffu, v, o);
      if (lane >= o) v += got;
    }
    if (b < p.B) prefix[b + 1] = sum + v;
    sum += __shfl_sync(0xffffffffu, v, 31);
  }
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
  int items, ctas;                // CTAs that have work: at least two tiles each
  __device__ __forceinline__ void start(const LatentParams& p, const int* prefix) {
    items = (p.H + N - 1) / N;
    g = 0;
    end = 1;
    if (p.persistent) {
      total = static_cast<long long>(prefix[p.B]) * items;
      ctas = static_cast<int>(min(static_cast<long long>(gridDim.x), (total + 1) / 2));
      const int cta = min(static_cast<int>(blockIdx.x), ctas);
      g = ctas > 0 ? total * cta / ctas : 0;
      end = cta < ctas ? total * (cta + 1) / ctas : g;
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
      w.last_cta = static_cast<int>(((g - w.first + nt) * ctas - 1) / total);
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
    if (w.rows <= 0 || !taken(p, w.b)) return false;       // not persistent: nothing here
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

// one look at a barrier, without suspending
__device__ __forceinline__ bool mbar_test(uint64_t* bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred P;\n\t"
      "mbarrier.test_wait.parity.shared::cta.b64 P, [%1], %2;\n\t"
      "selp.b32 %0, 1, 0, P;\n\t}"
      : "=r"(ok)
      : "r"(smem_u32(bar)), "r"(parity)
      : "memory");
  return ok != 0;
}
// whether the predicate holds for any thread of the four softmax warps; a barrier for them
__device__ __forceinline__ bool any_of_128(bool v) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred P, Q;\n\t"
      "setp.ne.u32 P, %1, 0;\n\t"
      "bar.red.or.pred Q, 1, 128, P;\n\t"
      "selp.u32 %0, 1, 0, Q;\n\t}"
      : "=r"(r)
      : "r"(static_cast<uint32_t>(v))
      : "memory");
  return r != 0;
}
// box of a page: 64 columns x 8 tokens x slabs x 2
__device__ __forceinline__ void tma_load_page(void* dst, const CUtensorMap* map, uint64_t* bar, int group) {
  asm volatile(
      "cp.async.bulk.tensor.4d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %3, %3, %4}], [%2];"
      ::"r"(smem_u32(dst)), "l"(reinterpret_cast<uint64_t>(map)), "r"(smem_u32(bar)), "r"(0), "r"(group)
      : "memory");
}

template <int N, int OG>
__global__ void __launch_bounds__(256 + 128 * OG, 1)
latent_attention_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const LatentParams p) {
  constexpr int W = N < 32 ? N : 32;            // columns per TMEM load
  constexpr int C = W / 2, NC = N / W;          // columns of a load that a softmax thread works on, loads per tile
  constexpr int NB = N == 64 ? 1 : 2;           // blocks of 128 value columns per output warp group
  extern __shared__ __align__(1024) uint8_t smem[];
  if ((smem_u32(smem) & 1023u) != 0u) {         // uniform over the CTA, before anything is allocated
    if (threadIdx.x == 0) report(p.status, kErrSmemLayout);
    return;
  }
  const int blocks = (p.value_slabs + 1) / 2, tile_bytes = p.slabs * kKeys * 128, group_bytes = p.slabs * 1024;
  uint8_t* sK = smem;                           // [stage][group of 8 keys][slab][8 x 128 bytes]
  uint8_t* sQ = sK + p.stages * tile_bytes;     // [slab][N rows of 128 bytes]
  uint8_t* sP = sQ + p.slabs * N * 128;         // [2][key][64 columns]
  float* s_max = reinterpret_cast<float*>(sP + 2 * kPTile);       // [4][N] maxima (sums) of the softmax warps
  float* s_m = s_max + 4 * N;                   // [N]
  float* s_alpha = s_m + N;                     // [2][N]
  float* s_l = s_alpha + 2 * N;                 // [N] factor of the output
  int* s_lo = reinterpret_cast<int*>(s_l + N);  // [N] first and last visible key of a row
  int* s_hi = s_lo + N;
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_hi + N);
  uint64_t* k_full = bars;                      // [kMaxStages]
  uint64_t* k_free = k_full + kMaxStages;       // [kMaxStages]
  uint64_t* s_full = k_free + kMaxStages;       // [2]
  uint64_t* p_ready = s_full + 2;               // [2]
  uint64_t* o_full = p_ready + 2;               // [2]
  uint64_t* o_free = o_full + 2;                // [2]
  uint64_t* q_full = o_free + 2;
  uint64_t* q_free = q_full + 1;
  uint64_t* l_ready = q_full + 2;
  uint64_t* l_free = q_full + 3;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(q_full + 4);
  int* s_rescale = reinterpret_cast<int*>(tmem_holder + 1);       // [2] a tile's s_alpha are not all 1
  int* prefix = reinterpret_cast<int*>(tmem_holder + 4);          // [B + 1], persistent only

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  uint32_t cols = 32;
  while (static_cast<int>(cols) < 2 * N * (1 + blocks)) cols <<= 1;
  if (threadIdx.x == 0) {
    for (int i = 0; i < kMaxStages; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_free[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&p_ready[i], 4);
      mbar_init(&o_full[i], 1);
      mbar_init(&o_free[i], 4 * OG);
    }
    mbar_init(q_full, 1);
    mbar_init(q_free, 1);
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
  if (p.persistent) {
    decode_tiles(p, prefix);
    __syncthreads();
    if (warp == 2) decode_prefix(p, prefix, lane);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tS = *tmem_holder, tO = tS + 2 * N;       // S^T: two buffers of N columns, O^T: two of `blocks` x N
  Waiter wait{p.status, false};
  Walk<N> walk;
  walk.start(p, prefix);
  Piece w;
  int j = 0, np = 0;                            // tiles and pieces so far

  if (warp == 0) {
    // ---------------- TMA producer ----------------
    bool ok = true;
    int stage = 0, round = 0;                   // of tile j
    while (ok && walk.next(p, prefix, w)) {
      for (int i = 0; i < w.tiles && ok; ++i, ++j) {
        const int page = (w.t_lo + (w.first + i) * kKeys) / kPage + (lane & 3);
        int blk = 0;
        if (page < p.max_blocks) blk = p.block_tables[static_cast<size_t>(w.b) * p.max_blocks + page];
        blk = min(max(blk, 0), p.num_blocks - 1);          // pages past the sequence are masked later
        if (i == 0) {
          if (np > 0) ok = wait(q_free, (np - 1) & 1, kErrProducerWait);
          ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
          if (!ok) break;
          if (lane == 0) mbar_arrive_expect_tx(q_full, p.slabs * N * 128);
          __syncwarp();
          if (lane < p.slabs) tma_load_2d(sQ + lane * N * 128, &tmQ, q_full, lane * 64, w.q_row);
        }
        if (round > 0) ok = wait(&k_free[stage], (round - 1) & 1, kErrProducerWait);
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (!ok) break;
        if (lane == 0) mbar_arrive_expect_tx(&k_full[stage], tile_bytes);
        __syncwarp();
        if (lane < 4) tma_load_page(sK + stage * tile_bytes + lane * 2 * group_bytes, &tmK, &k_full[stage], 2 * blk);
        if (++stage == p.stages) stage = 0, ++round;
      }
      ++np;
    }
    // copies in flight must land before the CTA's shared memory goes away
    if (lane == 0) {
      for (int s = 0; s < p.stages; ++s) {
        const int uses = round + (s < stage ? 1 : 0);
        if (uses > 0) mbar_wait(&k_full[s], (uses - 1) & 1);
      }
      if (np > 0) mbar_wait(q_full, (np - 1) & 1);
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (elect_one()) {
      constexpr uint32_t id = (1u << 4) | (1u << 7) | (1u << 10) | ((static_cast<uint32_t>(N) >> 3) << 17);
      constexpr uint32_t id_s = id | ((64u >> 4) << 24), id_o = id | ((128u >> 4) << 24) | (1u << 15) | (1u << 16);    // O^T: both MN-major
      const uint32_t q_addr = smem_u32(sQ), k_addr = smem_u32(sK), p_addr = smem_u32(sP);
      bool ok = true, more;
      int i = 0, stage = 0, round = 0, o_stage = 0;        // S^T: tile of the piece w, its stage; O^T: its stage
      auto next_tile = [&]() {
        if (j > 0 || np > 0) {
          ++i;
          if (++stage == p.stages) stage = 0, ++round;
          if (i < w.tiles) return true;
        }
        i = 0;
        ++np;                                              // pieces begun
        return walk.next(p, prefix, w);
      };
      auto landed = [&]() { return mbar_test(&k_full[stage], round & 1) && (i > 0 || mbar_test(q_full, (np - 1) & 1)); };
      auto issue_s = [&](int tile) {
        if (i == 0 && !wait(q_full, (np - 1) & 1, kErrMmaWaitFull)) return false;
        if (!wait(&k_full[stage], round & 1, kErrMmaWaitFull)) return false;
        tc_fence_after();
        const uint32_t d = tS + (tile & 1) * N;
        uint64_t da = make_desc(k_addr + stage * tile_bytes, 16, group_bytes), db = make_desc(q_addr, 16, 1024);
        for (int x = 0; x < p.slabs; ++x, da += 1024 >> 4, db += N * 128 >> 4) {
#pragma unroll
          for (int k = 0; k < 4; ++k)                      // 16 columns (32 bytes) per MMA
            mma_f16(d, da + (k * 32 >> 4), db + (k * 32 >> 4), id_s, x > 0 || k > 0 ? 1u : 0u);
        }
        tc_commit(&s_full[tile & 1]);
        if (i + 1 == w.tiles) tc_commit(q_free);
        return true;
      };
      more = next_tile();
      if (more) ok = issue_s(0);
      while (more && ok) {
        uint64_t* ready = &p_ready[j & 1];
        const uint32_t phase = (j >> 1) & 1;
        more = next_tile();
        bool issued = false;
        if (more) {
          for (uint32_t polls = 0; polls < (1u << 22) && !issued; ++polls) {
            if (landed()) {
              ok = issue_s(j + 1);
              issued = true;
            } else if (mbar_test(ready, phase)) {
              break;
            }
          }
        }
        if (!ok || !wait(ready, phase, kErrMmaWaitFull)) break;
        tc_fence_after();
        const uint32_t d = tO + (j & 1) * blocks * N;
        uint64_t da = make_desc(k_addr + o_stage * tile_bytes, 1024, group_bytes);
        const uint64_t db = make_desc(p_addr + (j & 1) * kPTile, 16, 1024);
        for (int x = 0; x < blocks; ++x, da += 2048 >> 4) {
#pragma unroll
          for (int k = 0; k < 4; ++k)                      // 16 keys per MMA: two groups of eight rows
            mma_f16(d + x * N, da + (2 * k * group_bytes >> 4), db + (k * 2048 >> 4), id_o, k > 0 ? 1u : 0u);
        }
        tc_commit(&o_full[j & 1]);
        tc_commit(&k_free[o_stage]);
        if (++o_stage == p.stages) o_stage = 0;
        if (more && !issued) ok = issue_s(j + 1);
        ++j;
      }
    }
  } else if (warp >= 4 && warp < 8) {
    // ---------------- softmax: a key and half of the columns of every load per thread ----------------
    const int quarter = warp & 3, tid = quarter * 32 + lane, half = lane >> 4, key = quarter * 16 + (lane & 15);
    const uint32_t addr = tS + (static_cast<uint32_t>(quarter * 32) << 16);       // rows 16 q .. 16 q + 15 in the first 16 lanes
    while (walk.next(p, prefix, w)) {
      float l[NC][C];
#pragma unroll
      for (int x = 0; x < NC; ++x)
#pragma unroll
        for (int c = 0; c < C; ++c) l[x][c] = 0.f;
      float m = kNoMax;                                    // thread c < N: reference maximum of row c
      if (tid < N) {
        s_m[tid] = kNoMax;
        const int pos = w.pos0 + (w.row0 % p.H + min(tid, w.rows - 1)) / p.H;
        s_lo[tid] = first_visible(pos, p.window);
        s_hi[tid] = pos;
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      // keys that every row sees
      const int lo_all = first_visible(w.pos1, p.window), hi_all = w.pos0;
      for (int i = 0; i < w.tiles; ++i, ++j) {
        const int buf = j & 1;
        const int t0 = w.t_lo + (w.first + i) * kKeys, t = t0 + key;
        const bool plain = t0 >= lo_all && t0 + kKeys - 1 <= hi_all;
        wait(&s_full[buf], (j >> 1) & 1, kErrEpilogueWait);
        tc_fence_after();
        float x[NC][C];
        bool over = false;
#pragma unroll
        for (int n = 0; n < NC; ++n) {
          float v[W];
          tmem_load<W>(addr + buf * N + n * W, v);
          const int col0 = n * W + half * C;
#pragma unroll
          for (int c = 0; c < C; ++c) {                    // the upper lanes take over the second half of the columns
            const float got = __shfl_xor_sync(0xffffffffu, v[c + C], 16);
            x[n][c] = (half ? got : v[c]) * p.scale_log2;
          }
          if (!plain) {
#pragma unroll
            for (int c = 0; c < C; ++c)
              if (t < s_lo[col0 + c] || t > s_hi[col0 + c]) x[n][c] = -INFINITY;
          }
#pragma unroll
          for (int c = 0; c < C; c += 4) {
            const float4 mm = *reinterpret_cast<const float4*>(s_m + col0 + c);
            over |= fmaxf(fmaxf(x[n][c] - mm.x, x[n][c + 1] - mm.y), fmaxf(x[n][c + 2] - mm.z, x[n][c + 3] - mm.w)) > kSlack;
          }
        }
        // the output of the tile before the last has been taken: its factors and its P^T are free
        if (j > 1) wait(&o_free[buf], ((j >> 1) - 1) & 1, kErrEpilogueWait);
        const bool rescale = any_of_128(over);
        if (tid == 0) s_rescale[buf] = rescale;
        if (rescale) {                                     // uniform over the four warps
#pragma unroll
          for (int n = 0; n < NC; ++n) {
            float y[C];
#pragma unroll
            for (int c = 0; c < C; ++c) y[c] = x[n][c];
            const float mx = column_reduce<C, false>(y, lane);
            if ((lane & 15) < C) s_max[quarter * N + n * W + half * C + (lane & 15)] = mx;
          }
          asm volatile("bar.sync 1, 128;" ::: "memory");
          if (tid < N) {
            const float mn = fmaxf(fmaxf(fmaxf(s_max[tid], s_max[N + tid]), fmaxf(s_max[2 * N + tid], s_max[3 * N + tid])), m);
            s_alpha[buf * N + tid] = ex2(m - mn);
            s_m[tid] = m = mn;
          }
          asm volatile("bar.sync 1, 128;" ::: "memory");
#pragma unroll
          for (int n = 0; n < NC; ++n)
#pragma unroll
            for (int c = 0; c < C; ++c) l[n][c] *= s_alpha[buf * N + n * W + half * C + c];
        }
        uint8_t* row = sP + buf * kPTile + key * 128;
#pragma unroll
        for (int n = 0; n < NC; ++n) {
          const int col0 = n * W + half * C;
#pragma unroll
          for (int c = 0; c < C; c += 8) {
            uint32_t packed[4];
#pragma unroll
            for (int e = 0; e < 8; e += 4) {
              const float4 mm = *reinterpret_cast<const float4*>(s_m + col0 + c + e);
              float* xs = &x[n][c + e];
              float* ls = &l[n][c + e];
              const float pr[4] = {ex2(xs[0] - mm.x), ex2(xs[1] - mm.y), ex2(xs[2] - mm.z), ex2(xs[3] - mm.w)};
              ls[0] += pr[0]; ls[1] += pr[1]; ls[2] += pr[2]; ls[3] += pr[3];
              const __nv_bfloat162 lo = __floats2bfloat162_rn(pr[0], pr[1]), hi = __floats2bfloat162_rn(pr[2], pr[3]);
              packed[e / 2] = *reinterpret_cast<const uint32_t*>(&lo);
              packed[e / 2 + 1] = *reinterpret_cast<const uint32_t*>(&hi);
            }
            *reinterpret_cast<uint4*>(row + ((((col0 + c) >> 3) ^ (key & 7)) << 4)) = make_uint4(packed[0], packed[1], packed[2], packed[3]);
          }
        }
        fence_proxy_async();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_ready[buf]);
      }
      // sums over the keys; what the output is multiplied by
#pragma unroll
      for (int n = 0; n < NC; ++n) {
        const float sum = column_reduce<C, true>(l[n], lane);
        if ((lane & 15) < C) s_max[quarter * N + n * W + half * C + (lane & 15)] = sum;
      }
      if (np > 0) wait(l_free, (np - 1) & 1, kErrEpilogueWait);
      asm volatile("bar.sync 1, 128;" ::: "memory");
      if (tid < N) {
        const float sum = (s_max[tid] + s_max[N + tid]) + (s_max[2 * N + tid] + s_max[3 * N + tid]);
        float f = 1.f;
        if (w.part < 0) {
          if (p.persistent && tid == 0) p.range[2 * w.item] = p.range[2 * w.item + 1] = 0;
          f = sum > 0.f ? 1.f / (sum + sink_term(p.sink, (w.q_row + tid) % p.H, m)) : 0.f;
          if (p.gate != nullptr && tid < w.rows) {
            const int row = w.q_row + tid;
            f *= __fdividef(1.f, 1.f + __expf(-__bfloat162float(p.gate[static_cast<long long>(row / p.H) * p.ld_gate + row % p.H])));
          }
        } else {
          if (tid == 0 && w.first == 0) {
            p.range[2 * w.item] = blockIdx.x;
            p.range[2 * w.item + 1] = w.last_cta;
          }
          float* ml = p.part_ml + (static_cast<size_t>(2 * blockIdx.x + w.part) * N + tid) * 2;
          ml[0] = m;
          ml[1] = sum;
        }
        s_l[tid] = f;
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
        const int buf = j & 1;
        wait(&o_full[buf], (j >> 1) & 1, kErrEpilogueWait);
        tc_fence_after();
        const bool rescale = s_rescale[buf] != 0;
#pragma unroll
        for (int x = 0; x < NB; ++x) {
          const int b = group + OG * x;
          if (b >= blocks) break;                          // warp-uniform
#pragma unroll
          for (int c0 = 0; c0 < N; c0 += W) {
            float v[W];
            tmem_load<W>(addr + (buf * blocks + b) * N + c0, v);
            if (rescale) {
#pragma unroll
              for (int c = 0; c < W; c += 4) {
                const float4 al = *reinterpret_cast<const float4*>(s_alpha + buf * N + c0 + c);
                o[x][c0 + c] *= al.x; o[x][c0 + c + 1] *= al.y; o[x][c0 + c + 2] *= al.z; o[x][c0 + c + 3] *= al.w;
              }
            }
#pragma unroll
            for (int c = 0; c < W; ++c) o[x][c0 + c] += v[c];
          }
        }
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&o_free[buf]);
      }
      wait(l_ready, np & 1, kErrEpilogueWait);
      float* part = p.part_o + static_cast<size_t>(2 * blockIdx.x + max(w.part, 0)) * N * p.out_cols;
#pragma unroll
      for (int x = 0; x < NB; ++x) {
        const int col0 = (group + OG * x) * 128 + quarter * 32;
        if (col0 >= p.out_cols) continue;                  // warp-uniform: a multiple of 64 columns
        if (w.part < 0) {
          // neighbouring lanes swap columns of two rows: an even lane stores the first row's pair, an odd one the second's
          __nv_bfloat162* dst = reinterpret_cast<__nv_bfloat162*>(p.out + static_cast<size_t>(w.q_row + (lane & 1)) * p.out_cols + col0 + (lane & ~1));
#pragma unroll
          for (int c = 0; c < N; c += 2) {
            const float a = o[x][c] * s_l[c], b = o[x][c + 1] * s_l[c + 1];
            const float got = __shfl_xor_sync(0xffffffffu, lane & 1 ? a : b, 1);
            if (c + (lane & 1) < w.rows) dst[static_cast<size_t>(c) * p.out_cols / 2] = lane & 1 ? __floats2bfloat162_rn(got, b) : __floats2bfloat162_rn(a, got);
          }
        } else {
          float* dst = part + col0 + lane;
#pragma unroll
          for (int c = 0; c < N; ++c)
            if (c < w.rows) dst[static_cast<size_t>(c) * p.out_cols] = o[x][c];
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

// Items of a persistent launch that several CTAs shared.  Grid (items, query rows), a block of 128 threads per row.
template <int N>
__global__ void __launch_bounds__(128)
latent_merge_kernel(const LatentParams p) {
  tgi::pdl_wait();
  tgi::pdl_trigger();
  constexpr int kBatch = 128;                              // parts whose weights are held at a time
  __shared__ float s_f[kBatch];
  __shared__ float red[8];
  const int items = (p.H + N - 1) / N, b = blockIdx.x / items, row = blockIdx.x % items * N + blockIdx.y, r = blockIdx.y;
  const int begin = p.cu[b];
  if (row >= p.H || !taken(p, b)) return;
  const int c0 = p.range[2 * blockIdx.x], c1 = p.range[2 * blockIdx.x + 1];
  if (c0 == c1) return;                                    // one CTA did the whole item
  // the first of the CTAs ended with its part (slot 1), the others began with theirs (slot 0)
  auto slot = [&](int c) { return static_cast<size_t>(2 * c + (c == c0 ? 1 : 0)) * N + r; };
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float mm = -INFINITY;
  for (int c = c0 + threadIdx.x; c <= c1; c += blockDim.x) mm = fmaxf(mm, p.part_ml[slot(c) * 2]);
#pragma unroll
  for (int o = 16; o; o >>= 1) mm = fmaxf(mm, __shfl_xor_sync(0xffffffffu, mm, o));
  if (lane == 0) red[warp] = mm;
  __syncthreads();
  mm = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
  float sum = 0.f;
  constexpr int kCols = 4;                                 // columns per thread: out_cols <= 512
  float o[kCols] = {};
  for (int at = c0; at <= c1; at += kBatch) {
    const int n = min(kBatch, c1 + 1 - at);
    __syncthreads();
    if (static_cast<int>(threadIdx.x) < n) {
      const float* ml = p.part_ml + slot(at + threadIdx.x) * 2;
      const float f = exp2f(ml[0] - mm);
      s_f[threadIdx.x] = f;
      sum = fmaf(ml[1], f, sum);
    }
    __syncthreads();
#pragma unroll 8
    for (int i = 0; i < n; ++i) {
      const float* src = p.part_o + slot(at + i) * p.out_cols;
      const float f = s_f[i];
#pragma unroll
      for (int e = 0; e < kCols; ++e) {
        const int col = threadIdx.x + e * 128;
        if (col < p.out_cols) o[e] = fmaf(src[col], f, o[e]);
      }
    }
  }
#pragma unroll
  for (int d = 16; d; d >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
  if (lane == 0) red[4 + warp] = sum;
  __syncthreads();
  sum = (red[4] + red[5]) + (red[6] + red[7]);
  float f = sum > 0.f ? 1.f / (sum + sink_term(p.sink, row, mm)) : 0.f;
  if (p.gate != nullptr)
    f *= __fdividef(1.f, 1.f + __expf(-__bfloat162float(p.gate[static_cast<long long>(begin) * p.ld_gate + row])));
#pragma unroll
  for (int e = 0; e < kCols; ++e) {
    const int col = threadIdx.x + e * 128;
    if (col < p.out_cols) p.out[(static_cast<size_t>(begin) * p.H + row) * p.out_cols + col] = __float2bfloat16(o[e] * f);
  }
}

int smem_bytes(int N, int slabs, int stages, int seqs) {
  return stages * slabs * kKeys * 128 + slabs * N * 128 + 2 * kPTile + 10 * N * 4 + (2 * kMaxStages + 12) * 8 + 16 + (seqs + 1) * 4;
}
// stages of the K ring that fit (at least two are wanted)
int stages_for(int N, int slabs) {
  int n = kMaxStages;
  while (n > 0 && smem_bytes(N, slabs, n, kMaxSeqs) > 227 * 1024) --n;
  return n;
}
// map over pages [num_blocks, 16, slabs * 64] whose box is one page: 64 columns x 8 tokens x slabs x 2
int make_page_map(CUtensorMap* map, const void* pages, int num_blocks, int slabs) {
  tgi::EncodeTiledFn enc = tgi::get_encode();
  if (enc == nullptr) return -100;
  const cuuint64_t row = static_cast<cuuint64_t>(slabs) * 128;
  cuuint64_t dims[4] = {64, 8, static_cast<cuuint64_t>(slabs), 2 * static_cast<cuuint64_t>(num_blocks)};
  cuuint64_t strides[3] = {row, 128, 8 * row};
  cuuint32_t box[4] = {64, 8, static_cast<cuuint32_t>(slabs), 2}, step[4] = {1, 1, 1, 1};
  const CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(pages), dims, strides, box, step,
                         CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                         CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -static_cast<int>(r) - 1000;
}

template <int N, int OG>
int launch(const LatentParams& p, const void* q, const void* pages, long long q_rows, int max_q, int ctas, cudaStream_t stream) {
  CUtensorMap tmQ, tmK;
  const uint64_t width = static_cast<uint64_t>(p.slabs) * 64;
  int rc = tgi::make_map_2d(&tmQ, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, q, q_rows, width, width * 2, N, 64, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  rc = make_page_map(&tmK, pages, p.num_blocks, p.slabs);
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
  const size_t smem = smem_bytes(N, p.slabs, p.stages, p.persistent ? p.B : 0);
  tgi::launch(kern, grid, dim3(256 + 128 * OG), smem, stream, tmQ, tmK, p);
  if (p.persistent) tgi::launch(latent_merge_kernel<N>, dim3(p.B * items, min(N, p.H)), dim3(128), 0, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace

extern "C" {

// Query rows per tile for rows of `slabs` x 64 columns, `value_slabs` of them values; 0: the kernel does not take them.
int tgi_latent_rows(int slabs, int value_slabs, long long rows) {
  if (value_slabs < 1 || value_slabs > 8 || slabs < value_slabs || slabs > kMaxSlabs) return 0;
  int N = rows <= 16 ? 16 : rows <= 32 || value_slabs > 4 ? 32 : 64;
  while (N >= 16 && stages_for(N, slabs) < 2) N /= 2;
  return N >= 16 ? N : 0;
}

// q [T, H, slabs * 64] and pages [num_blocks, 16, slabs * 64] bf16 (the first value_slabs * 64 columns of a row are the
// values), out [T, H, value_slabs * 64]; no sequence brings more than max_q tokens.  part_o / part_ml: 2 * ctas slots of N x (value_slabs * 64) and N x 2 floats, range:
// 2 * B * ceil(H / N) ints; used when max_q == 1.  Sequences whose entry in `elsewhere` (optional, [B]) is at
// least their number of tokens are left out (and may bring more than max_q).  gate (optional): [T, ld_gate]; sink (optional): [H].
int tgi_latent_attention(const void* q, const void* pages, const int* block_tables, const int* cu, const int* kv_lens,
                         const void* gate, long long ld_gate, const float* sink, void* out, float* part_o, float* part_ml, int* range, int T, int B, int max_q,
                         int max_blocks, int num_blocks, int H, int slabs, int value_slabs, int N, float scale, int window,
                         const int* elsewhere, int ctas, int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || max_q <= 0) return 0;
  if (N != 16 && N != 32 && N != 64) return -10;
  if (B > 65535 || num_blocks < 1 || max_blocks < 1 || ctas < 1 || slabs > kMaxSlabs || value_slabs > 8 ||
      stages_for(N, slabs) < 2)
    return -10;
  LatentParams p;
  p.block_tables = block_tables;
  p.cu = cu;
  p.kv_lens = kv_lens;
  p.gate = static_cast<const __nv_bfloat16*>(gate);
  p.ld_gate = ld_gate;
  p.sink = sink;
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
  p.stages = stages_for(N, slabs);
  p.window = window;
  p.persistent = max_q == 1 && B <= kMaxSeqs && part_o != nullptr && part_ml != nullptr && range != nullptr;
  p.elsewhere = elsewhere;
  p.scale_log2 = scale * kLog2e;
  p.status = status;
  const long long rows = static_cast<long long>(T) * H;
  const bool wide = value_slabs > 4;
  if (N == 64) return wide ? -10 : launch<64, 2>(p, q, pages, rows, max_q, ctas, stream);
  if (N == 32) return wide ? launch<32, 2>(p, q, pages, rows, max_q, ctas, stream) : launch<32, 1>(p, q, pages, rows, max_q, ctas, stream);
  return wide ? launch<16, 2>(p, q, pages, rows, max_q, ctas, stream) : launch<16, 1>(p, q, pages, rows, max_q, ctas, stream);
}

}  // extern "C"
