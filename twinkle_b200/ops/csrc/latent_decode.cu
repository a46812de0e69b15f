// Latent decode attention on the tensor cores: one query token per sequence, all heads against the same cached rows (bf16).
//
// The cached rows of a sequence are key and value of every head, so a tile of 128 tokens × rank is brought into shared memory
// once and used by two products with the tokens (or the rank) on the 128 rows of the tensor core and the heads as columns:
//     Sᵀ [tokens, heads] = C · Qᵀ                 C as it lies: tokens are rows, the rank is reduced
//     Oᵀ [rank, heads]  += Cᵀ · Pᵀ                the same shared memory read the other way round: tokens are reduced
// Heads need not fill a 128-row tile, which a product with heads as rows would leave mostly empty.  A row's value is its first R columns;
// rotated key dimensions behind them enter the first product only.  With a window the tiles start at the first token it reaches.
//
// One CTA per (part of the context, group of up to 64 heads, sequence), 192 threads:
//   warps 0-3  softmax: thread = one token; maxima over tokens by a transposing butterfly in each warp, then over warps; weights go
//              to shared memory as bf16; the accumulator is rescaled only when a maximum grows by more than 2^8.  Epilogue.
//   warp 4     producer: queries once, then pieces of 128 tokens × 128 of the rank; every page of the table is one TMA box per 64
//              columns, issued by a lane of its own
//   warp 5     issues the products
// Tensor memory: Sᵀ in two buffers [0, 128), Oᵀ in pieces of 128 ranks from column 128 on.  Parts of a context leave their sums,
// maxima and results to a small combining kernel.  The sink logit starts the running maximum; the first part counts it.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"

namespace tk {

using bf16 = __nv_bfloat16;
using OptT = c10::optional<torch::Tensor>;

namespace ld {
constexpr int TT = 128;                       // tokens per tile
constexpr int CHUNK = TT * 64 * 2;            // 64 columns of a tile
constexpr int PIECE = 2 * CHUNK;              // 128 columns: the unit of the ring
constexpr int MAX_RING = 6, MAX_VALUE_PIECES = 4;
constexpr float FAR = -1e30f;                 // running maximum before the first score
constexpr int THREADS = 192;
constexpr float RESCALE = 8.f;                // log2 units
constexpr float LOG2E = 1.4426950408889634f;
constexpr int BARS = 1024;                    // barriers and small arrays
}  // namespace ld

struct LatentDecode {
  const int* tables;
  const int* lens;
  const bf16* sinks;
  const bf16* gate; long ldg;
  bf16* out;                                  // [B, H, R]; scores run over K ≥ R columns
  float *part_o, *part_m, *part_l;            // [parts, B, H, R], [parts, B, H] twice (parts > 1)
  int B, H, K, R, page, max_pages, parts, ring, window;
  float scale_log2;
  int* err;
};

struct OpMax { __device__ __forceinline__ float operator()(float a, float b) const { return fmaxf(a, b); } };
struct OpSum { __device__ __forceinline__ float operator()(float a, float b) const { return a + b; } };

// N values per lane → the reduction of value (lane mod N) over the 32 lanes, N = 16 or 32
template <int N, typename Op>
__device__ __forceinline__ float transposed_reduce(float (&v)[N], int lane, Op op) {
  if constexpr (N == 16) {
#pragma unroll
    for (int i = 0; i < 16; ++i) v[i] = op(v[i], __shfl_xor_sync(0xffffffffu, v[i], 16));
  }
#pragma unroll
  for (int o = N / 2; o > 0; o >>= 1) {
    const bool upper = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = upper ? v[i] : v[i + o], kept = upper ? v[i + o] : v[i];
      v[i] = op(kept, __shfl_xor_sync(0xffffffffu, send, o));
    }
  }
  return v[0];
}

template <int N>
__global__ void __launch_bounds__(ld::THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmC, const LatentDecode p) {
  using namespace ld;
  constexpr int W = N < 32 ? N : 32;          // heads per butterfly
  const int part = blockIdx.x, h0 = blockIdx.y * N, b = blockIdx.z;
  const int n = p.lens[b], lo = p.window > 0 ? max(0, n - p.window) : 0;
  const int tiles_all = (n + TT - 1) / TT - lo / TT, per = (tiles_all + p.parts - 1) / p.parts;
  const int first = lo / TT + part * per, tiles = max(0, min(tiles_all - part * per, per));
  const int pieces = (p.K + 127) / 128, value_pieces = (p.R + 127) / 128, ring = p.ring;

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* s_c = smem;                                    // [ring][2][128 tokens][64]
  uint8_t* s_q = s_c + ring * PIECE;                      // [2 · pieces][N][64]
  uint8_t* s_p = s_q + 2 * pieces * N * 128;              // [2][N][64 tokens]
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_p + 2 * N * 128);
  uint64_t *q_full = bars, *c_full = bars + 1, *c_empty = c_full + MAX_RING, *s_full = c_empty + MAX_RING, *s_empty = s_full + 2, *p_ready = s_empty + 2,
           *o_done = p_ready + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 1);
  int* s_any = reinterpret_cast<int*>(tmem_slot + 2);     // [2]
  float* s_m = reinterpret_cast<float*>(bars) + 64;       // [64] running maximum, [64] factor of this tile, [4][64] maxima / sums of the warps
  float *s_alpha = s_m + 64, *s_w = s_alpha + 64;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < ring; ++i) { mbar_init(&c_full[i], 1); mbar_init(&c_empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&s_full[i], 1); mbar_init(&s_empty[i], 128); }
    mbar_init(p_ready, 128);
    mbar_init(o_done, 1);
    fence_barrier_init();
  }
  if (threadIdx.x < N) s_m[threadIdx.x] = p.sinks == nullptr ? FAR : (h0 + static_cast<int>(threadIdx.x) < p.H ? __bfloat162float(p.sinks[h0 + threadIdx.x]) * LOG2E : 0.f);
  if (warp == 5) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(tmem_slot), tmem_o = tmem + 128;

  if (warp == 4) {
    // ------------------------------------------------------------- producer
    if (tiles > 0) {
      if (lane == 0) {
        tma_prefetch_desc(&tmQ);
        tma_prefetch_desc(&tmC);
        mbar_expect_tx(q_full, 2 * pieces * N * 128);
        for (int c = 0; c < 2 * pieces; ++c) tma_load_2d(s_q + c * N * 128, &tmQ, q_full, c * 64, b * p.H + h0);
      }
      const int pages = TT / p.page, last = (n + p.page - 1) / p.page;
      const int* table = p.tables + static_cast<size_t>(b) * p.max_pages;
      int slot = 0;
      uint32_t phase = 0;
      bool ok = true;
      for (int j = 0; ok && j < tiles; ++j) {
        const int pg = (first + j) * pages + lane;
        // places past the end of the sequence read page 0: finite rows whose weight is zero
        const int row = lane < pages && pg < last ? table[pg] * p.page : 0;
        for (int c = 0; c < pieces; ++c) {
          ok = mbar_wait(&c_empty[slot], phase ^ 1, p.err, ERR_PRODUCER_WAIT);
          if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
          if (lane == 0) mbar_expect_tx(&c_full[slot], PIECE);
          __syncwarp();
          if (lane < pages) {
            uint8_t* dst = s_c + slot * PIECE + lane * p.page * 128;
            tma_load_2d(dst, &tmC, &c_full[slot], c * 128, row);
            tma_load_2d(dst + CHUNK, &tmC, &c_full[slot], c * 128 + 64, row);
          }
          if (++slot == ring) { slot = 0; phase ^= 1; }
        }
      }
      if (!ok) for (int s = 0; s < ring; ++s) mbar_wait(&c_full[s], 0, nullptr, 0);   // copies in flight get a bounded chance to land
    }
  } else if (warp == 5) {
    // ----------------------------------------------------------- products
    if (lane == 0 && tiles > 0) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(128, N, false, false), idesc_o = umma_idesc_bf16(128, N, true, false);
      const uint32_t a_c = smem_u32(s_c), a_q = smem_u32(s_q), a_p = smem_u32(s_p);
      int slot = 0, o_slot = 0;
      uint32_t phase = 0;
      bool ok = mbar_wait(q_full, 0, p.err, ERR_ATTN_WAIT);
      auto scores = [&](int j) {
        if (j >= 2 && !mbar_wait(&s_empty[j & 1], ((j >> 1) - 1) & 1, p.err, ERR_ATTN_WAIT)) { ok = false; return; }
        for (int c = 0; c < pieces; ++c) {
          if (!mbar_wait(&c_full[slot], phase, p.err, ERR_ATTN_WAIT)) { ok = false; return; }
          tc_fence_after();
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            const uint32_t in = (k & 3) * 32;
            umma_bf16(tmem + (j & 1) * 64, umma_desc(a_c + slot * PIECE + (k >> 2) * CHUNK + in, 16, 1024), umma_desc(a_q + (2 * c + (k >> 2)) * N * 128 + in, 16, 1024),
                      idesc_s, c > 0 || k > 0 ? 1u : 0u);
          }
          if (++slot == ring) { slot = 0; phase ^= 1; }
        }
        umma_commit(&s_full[j & 1]);
      };
      const bool ahead = ring >= 2 * pieces;              // room for the next tile beside this one
      if (ok) scores(0);
      for (int j = 0; ok && j < tiles; ++j) {
        if (ahead && j + 1 < tiles) scores(j + 1);
        if (ok) ok = mbar_wait(p_ready, j & 1, p.err, ERR_ATTN_WAIT);
        if (!ok) break;
        tc_fence_after();
        for (int c = 0; c < pieces; ++c) {
          if (c < value_pieces) {
#pragma unroll
            for (int k = 0; k < TT / 16; ++k)
              umma_bf16(tmem_o + c * N, umma_desc(a_c + o_slot * PIECE + k * 2048, CHUNK, 1024), umma_desc(a_p + (k >> 2) * N * 128 + (k & 3) * 32, 16, 1024), idesc_o,
                        j > 0 || k > 0 ? 1u : 0u);
          }
          umma_commit(&c_empty[o_slot]);
          if (++o_slot == ring) o_slot = 0;
        }
        umma_commit(o_done);
        if (!ahead && j + 1 < tiles) scores(j + 1);
      }
    }
  } else {
    // -------------------------------------------------------------- softmax
    const int t = threadIdx.x;                            // token of the tile == TMEM lane
    const uint32_t lanes = static_cast<uint32_t>(warp * 32) << 16;
    float l[N];
#pragma unroll
    for (int i = 0; i < N; ++i) l[i] = 0.f;
    bool dead = false;
    for (int j = 0; j < tiles; ++j) {
      float s[N];
      if (!dead && !mbar_wait(&s_full[j & 1], (j >> 1) & 1, p.err, ERR_ATTN_WAIT)) dead = true;
      if (!dead) {
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < (N + 31) / 32; ++c) {
          uint32_t r[32];
          tmem_ld32(tmem + (j & 1) * 64 + c * 32 + lanes, r);      // N = 16: columns 16-31 are not used
          tmem_ld_wait();
          const int at = (first + j) * TT + t;
          const bool live = at < n && at >= lo;
#pragma unroll
          for (int i = 0; i < W; ++i) s[c * 32 + i] = live ? __uint_as_float(r[i]) * p.scale_log2 : -INFINITY;
        }
        tc_fence_before();
        mbar_arrive(&s_empty[j & 1]);
      } else {
#pragma unroll
        for (int i = 0; i < N; ++i) s[i] = 0.f;
      }
#pragma unroll
      for (int c = 0; c < N / W; ++c) {
        float v[W];
#pragma unroll
        for (int i = 0; i < W; ++i) v[i] = s[c * W + i];
        const float m = transposed_reduce<W>(v, lane, OpMax());
        if (lane < W) s_w[warp * 64 + c * W + lane] = m;
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      if (t < (N < 32 ? 32 : N)) {
        bool grows = false;
        if (t < N) {
          const float m = fmaxf(fmaxf(s_w[t], s_w[64 + t]), fmaxf(s_w[128 + t], s_w[192 + t])), old = s_m[t];
          grows = m > old + RESCALE;
          s_alpha[t] = grows ? exp2f(old - m) : 1.f;
          if (grows) s_m[t] = m;
        }
        const bool any = __any_sync(0xffffffffu, grows);
        if (lane == 0) s_any[warp] = any;
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      const bool rescale = s_any[0] || (N > 32 && s_any[1]);
      // weights and accumulator are free once the products of the tile before have retired
      if (!dead && j > 0 && !mbar_wait(o_done, (j - 1) & 1, p.err, ERR_ATTN_WAIT)) dead = true;
      if (rescale) {
#pragma unroll
        for (int i = 0; i < N; ++i) l[i] *= s_alpha[i];
        if (!dead && j > 0) {
          tc_fence_after();
          for (int c = 0; c < value_pieces * N / W; ++c) {
            uint32_t r[32];
            const uint32_t at = tmem_o + c * W + lanes;
            tmem_ld32(at, r);                             // N = 16: the second half is the next piece's and goes back unchanged
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < W; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * s_alpha[(c * W) % N + i]);
            tmem_st32(at, r);
            tmem_st_wait();
          }
        }
      }
      uint8_t* row = s_p + (t >> 6) * (N * 128) + (t & 7) * 2;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const bf16 w = __float2bfloat16(fast_exp2(s[i] - s_m[i]));
        l[i] += __bfloat162float(w);                       // the sum of what the product will use
        *reinterpret_cast<bf16*>(row + i * 128 + ((((t & 63) >> 3) ^ (i & 7)) << 4)) = w;
      }
      tc_fence_before();
      fence_proxy_async();
      mbar_arrive(p_ready);
    }
    // ------------------------------------------------------------- epilogue
#pragma unroll
    for (int c = 0; c < N / W; ++c) {
      float v[W];
#pragma unroll
      for (int i = 0; i < W; ++i) v[i] = l[c * W + i];
      const float sum = transposed_reduce<W>(v, lane, OpSum());
      if (lane < W) s_w[warp * 64 + c * W + lane] = sum;
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    if (t < N && h0 + t < p.H) {
      float sum = s_w[t] + s_w[64 + t] + s_w[128 + t] + s_w[192 + t];
      if (part == 0 && p.sinks != nullptr) sum += exp2f(__bfloat162float(p.sinks[h0 + t]) * LOG2E - s_m[t]);
      const size_t at = (static_cast<size_t>(part) * p.B + b) * p.H + h0 + t;
      if (p.parts > 1) {
        p.part_m[at] = s_m[t];
        p.part_l[at] = sum;
      } else {
        float f = sum > 0.f ? 1.f / sum : 0.f;
        if (p.gate != nullptr) f /= 1.f + __expf(-__bfloat162float(p.gate[b * p.ldg + h0 + t]));
        s_alpha[t] = f;
      }
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    bool done = tiles == 0 || (!dead && mbar_wait(o_done, (tiles - 1) & 1, p.err, ERR_ATTN_WAIT));
    if (done) {
      tc_fence_after();
      for (int c = 0; c < value_pieces; ++c) {
        const int rank = c * 128 + t;
#pragma unroll
        for (int q = 0; q < N / W; ++q) {
          uint32_t r[32];
          if (tiles > 0) {
            tmem_ld32(tmem_o + c * N + q * W + lanes, r);
            tmem_ld_wait();
          } else {
#pragma unroll
            for (int i = 0; i < 32; ++i) r[i] = 0u;
          }
          if (rank < p.R) {
#pragma unroll
            for (int i = 0; i < W; ++i) {
              const int h = h0 + q * W + i;
              if (h < p.H) {
                if (p.parts > 1) p.part_o[((static_cast<size_t>(part) * p.B + b) * p.H + h) * p.R + rank] = __uint_as_float(r[i]);
                else p.out[(static_cast<size_t>(b) * p.H + h) * p.R + rank] = __float2bfloat16(__uint_as_float(r[i]) * s_alpha[q * W + i]);
              }
            }
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// One block per (head, sequence): parts weighed by their sums, each relative to the largest maximum.
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentDecode p) {
  const int h = blockIdx.x, b = blockIdx.y;
  const size_t at = static_cast<size_t>(b) * p.H + h, step = static_cast<size_t>(p.B) * p.H;
  float m = -INFINITY, l = 0.f;
  for (int s = 0; s < p.parts; ++s) m = fmaxf(m, p.part_m[s * step + at]);
  for (int s = 0; s < p.parts; ++s) l += p.part_l[s * step + at] * exp2f(p.part_m[s * step + at] - m);
  float f = l > 0.f ? 1.f / l : 0.f;
  if (p.gate != nullptr) f /= 1.f + __expf(-__bfloat162float(p.gate[b * p.ldg + h]));
  for (int r = threadIdx.x; r < p.R; r += 128) {
    float o = 0.f;
    for (int s = 0; s < p.parts; ++s) o += p.part_o[(s * step + at) * p.R + r] * exp2f(p.part_m[s * step + at] - m);
    p.out[at * p.R + r] = __float2bfloat16(o * f);
  }
}

// Whether the tensor-core form takes these operands; if so, runs it.
bool latent_decode_tc(const torch::Tensor& q, const torch::Tensor& pool, const torch::Tensor& tables, const torch::Tensor& lens, double scale, const OptT& sinks,
                      const OptT& gate, int window, torch::Tensor& out) {
  const int B = q.size(0), H = q.size(1), K = q.size(2), R = out.size(2), page = pool.size(1);
  if (q.scalar_type() != torch::kBFloat16 || K % 8 != 0 || R % 8 != 0 || R > 128 * ld::MAX_VALUE_PIECES || pool.size(3) != K || page < 8 || ld::TT % page != 0) return false;
  if (reinterpret_cast<uintptr_t>(q.data_ptr()) % 16 != 0 || reinterpret_cast<uintptr_t>(pool.data_ptr()) % 16 != 0 || B > 65535) return false;
  const int pieces = (K + 127) / 128;
  LatentDecode p{};
  int N = H <= 16 ? 16 : (H <= 32 ? 32 : 64), fixed = 0;
  for (;; N /= 2) {                     // rows too wide for 64 heads at a time: fewer heads per block
    fixed = 2 * pieces * N * 128 + 2 * N * 128 + 1024 + 4096;
    p.ring = std::min((227 * 1024 - fixed) / ld::PIECE, ld::MAX_RING);
    if (p.ring >= pieces || N == 16) break;
  }
  if (p.ring < pieces) return false;
  const int groups = (H + N - 1) / N;
  p.B = B; p.H = H; p.K = K; p.R = R; p.page = page; p.max_pages = tables.size(1); p.window = window;
  int most = (p.max_pages * page + ld::TT - 1) / ld::TT;
  if (window > 0) most = std::min(most, (window + ld::TT - 2) / ld::TT + 1);
  p.parts = std::max(1, std::min({most, num_sms() / (B * groups), 32}));
  p.tables = tables.data_ptr<int>(); p.lens = lens.data_ptr<int>();
  if (sinks.has_value() && sinks->defined()) p.sinks = reinterpret_cast<const bf16*>(sinks->data_ptr());
  if (gate.has_value() && gate->defined()) { p.gate = reinterpret_cast<const bf16*>(gate->data_ptr()); p.ldg = gate->stride(0); }
  p.out = reinterpret_cast<bf16*>(out.data_ptr());
  p.scale_log2 = static_cast<float>(scale) * ld::LOG2E;
  p.err = error_word();
  torch::Tensor po, pml;
  if (p.parts > 1) {
    auto f32 = q.options().dtype(torch::kFloat32);
    po = torch::empty({p.parts, B, H, R}, f32);
    pml = torch::empty({2, p.parts, B, H}, f32);
    p.part_o = po.data_ptr<float>(); p.part_m = pml.data_ptr<float>(); p.part_l = p.part_m + static_cast<size_t>(p.parts) * B * H;
  }
  CUtensorMap tq = make_tmap_2d(q.data_ptr(), K, static_cast<uint64_t>(B) * H, K, 64, N);
  CUtensorMap tc = make_tmap_2d(pool.data_ptr(), K, static_cast<uint64_t>(pool.size(0)) * page, K, 64, page);
  const int smem = p.ring * ld::PIECE + fixed;
  auto stream = at::cuda::getCurrentCUDAStream();
  auto go = [&](auto kern) {
    TK_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    kern<<<dim3(p.parts, groups, B), ld::THREADS, smem, stream>>>(tq, tc, p);
    count_launch();
    TK_CUDA_CHECK(cudaGetLastError());
  };
  if (N == 16) go(latent_decode_kernel<16>); else if (N == 32) go(latent_decode_kernel<32>); else go(latent_decode_kernel<64>);
  if (p.parts > 1) {
    latent_combine_kernel<<<dim3(H, B), 128, 0, stream>>>(p);
    count_launch();
    TK_CUDA_CHECK(cudaGetLastError());
  }
  return true;
}

}  // namespace tk
