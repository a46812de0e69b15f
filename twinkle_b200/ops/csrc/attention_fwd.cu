// Flash-attention forward for sm_100a: causal, GQA, packed variable-length sequences, query / key widths up to 192, value widths up to
// 128.  A row narrower than its tile of 64-wide chunks is filled up with zeros by the TMA load (the tensor map ends at the row's width).
// Optional: only the last `window` keys or the query's block of `chunk` positions (key blocks before them are not loaded), sink logits, a
// gate per head or element, score terms (TERMS: cap, factor per head, a number for the distance; the 255 distances of a tile are looked up or
// formed once per tile, one per softmax thread), and a last chunk of key dimensions that all heads share (rotated part of latent attention), loaded from a tensor of
// its own so that nothing has to put the keys together.
//
// One CTA per (128-row query tile of one sequence, query head).  192 threads:
//   warps 0-3  softmax: thread = one query row; reads S from tensor memory (tcgen05.ld), keeps the
//              running max / sum, writes P (bf16) into a 128-byte-swizzled smem tile, rescales the O
//              accumulator in tensor memory only when a row maximum grows by more than 2^8
//   warp 4     TMA producer: Q once, then K/V tiles (double buffered)
//   warp 5     MMA issuer: S_j = Q·K_jᵀ into one of two TMEM buffers (so S_{j+1} is computed while
//              the softmax of S_j runs), O += P_j·V_j into a third TMEM buffer
// Tensor memory: S0 [0,128), S1 [128,256), O [256,384) fp32 columns.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"
#include "scores.cuh"

namespace tk {

using bf16 = __nv_bfloat16;

namespace fa {
constexpr int BQ = 128, BKV = 128, D = 128;
constexpr int TILE_BYTES = 128 * 128 * 2;  // 32 KiB, two [128][64] swizzle atoms
constexpr int ATOM_BYTES = 128 * 64 * 2;   // 16 KiB
// Q and two stages of K of KA atoms each, V in two stages (one when three-atom keys leave no room for more), P, barriers
template <int KA>
struct Smem {
  static constexpr int K_TILE = KA > 2 ? 3 * ATOM_BYTES : TILE_BYTES, V_STAGES = KA > 2 ? 1 : 2;
  static constexpr int Q = 0, K = K_TILE, V = 3 * K_TILE, P = V + V_STAGES * TILE_BYTES, BAR = P + TILE_BYTES;
  static constexpr int XCHG = BAR + 256;            // row max (2 parities x 2 halves x 128) + row sums (2 x 128) floats
  static constexpr int BAND = XCHG + 6 * 128 * 4;   // numbers of the tile's distances, two tiles
  static constexpr int TOTAL = BAND + 2 * 256 * 4 + 1024;
};
constexpr int THREADS = 320;  // warps 0-7 softmax (two groups of 4: each owns 64 of the 128 S columns), 8 producer, 9 MMA
constexpr float RESCALE_THRESHOLD = 8.f;  // log2 units
}  // namespace fa

struct FwdParams {
  bf16* out;          // [T, Hq, D]
  float* lse;         // [Hq, T]  natural-log LSE of the scaled scores
  int e;              // width of a value / output row (a multiple of 8)
  const int* cu;      // [n+1] query boundaries
  const int* cu_k;    // [n+1] key/value boundaries (== cu for self-attention over the same packing)
  int T, hq, hkv;
  float scale_log2;   // softmax scale · log2(e)
  int causal;
  const bf16* sinks;  // [Hq] logit of a key without a value that every row sees (nullptr: none)
  OutGate gate;       // the output is multiplied by its sigmoid
  bool gate_vec;      // gates per element on 16-byte boundaries
  ScoreTerms terms;
  int window, chunk;  // what a query sees of the keys before it (0: no bound)
  int own_chunks;     // leading chunks of a key that are its head's own; the rest come from the shared tensor
  int tail_col;       // first column of a query row that meets the shared part
  int* err;
};

// KA / VA: 64-wide chunks of a query / key row (up to 3) and of a value row (1 or 2).
template <int KA, int VA, bool TERMS>
__global__ void __launch_bounds__(fa::THREADS, 1)
flash_fwd_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                 const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmR, const FwdParams p) {
  using namespace fa;
  using S = Smem<KA>;
  constexpr int VS = S::V_STAGES;
  const int head = blockIdx.x, seq = blockIdx.z;
  const int seq_start = p.cu[seq], seq_len = p.cu[seq + 1] - seq_start;
  // longest-first: the heaviest (last) query tiles are scheduled first
  const int n_qtiles = (seq_len + BQ - 1) / BQ;
  if (static_cast<int>(blockIdx.y) >= n_qtiles) return;
  const int qt = n_qtiles - 1 - blockIdx.y;
  const int q0 = qt * BQ;
  const int kv_head = head / (p.hq / p.hkv);
  // keys may be longer than queries (a query chunk against a key prefix): the causal diagonal is aligned to the
  // bottom-right corner, i.e. query row r sees keys 0 … r + q_off
  const int kv_start = p.cu_k[seq], kv_len = p.cu_k[seq + 1] - kv_start;
  const int q_off = kv_len - seq_len;
  const int kv_end = p.causal ? max(0, min(kv_len, q0 + BQ + q_off)) : kv_len;
  const bool bounded = p.window > 0 || p.chunk > 0;
  const int jb0 = bounded ? first_visible(max(q0 + q_off, 0), p.window, p.chunk) / BKV : 0;    // first key block that any row sees
  const int n_blocks = max(0, (kv_end + BKV - 1) / BKV - jb0);

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + S::BAR);
  uint64_t* q_full = bars;            // 1
  uint64_t* k_full = bars + 1;        // 2
  uint64_t* v_full = bars + 3;        // 2
  uint64_t* kv_empty = bars + 5;      // 2
  uint64_t* s_full = bars + 7;        // 2
  uint64_t* s_empty = bars + 9;       // 2
  uint64_t* p_ready = bars + 11;      // 1
  uint64_t* o_done = bars + 12;       // 1
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 13);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&kv_empty[i], 1);
      mbar_init(&s_full[i], 1);
      mbar_init(&s_empty[i], 256);
    }
    mbar_init(p_ready, 256);
    mbar_init(o_done, 1);
    fence_barrier_init();
  }
  if (warp == 9) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t*>(tmem_slot);
  const uint32_t tmem_o = tmem_base + 256;

  if (warp == 8) {
    // ------------------------------------------------------------- producer
    if (lane == 0) {
      tma_prefetch_desc(&tmQ);
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmV);
      mbar_expect_tx(q_full, KA * ATOM_BYTES);
#pragma unroll
      for (int c = 0; c < KA; ++c)
        tma_load_3d(smem + S::Q + c * ATOM_BYTES, &tmQ, q_full, c < p.own_chunks ? c * 64 : p.tail_col, head, seq_start + q0);
      for (int j = 0; j < n_blocks; ++j) {
        const int st = j & 1;
        if (j >= 2 && !mbar_wait(&kv_empty[st], ((j >> 1) - 1) & 1, p.err, ERR_ATTN_WAIT)) break;
        const int row = kv_start + (jb0 + j) * BKV;
        mbar_expect_tx(&k_full[st], KA * ATOM_BYTES);
#pragma unroll
        for (int c = 0; c < KA; ++c) {
          uint8_t* dst = smem + S::K + st * S::K_TILE + c * ATOM_BYTES;
          if (c < p.own_chunks) tma_load_3d(dst, &tmK, &k_full[st], c * 64, kv_head, row);
          else tma_load_3d(dst, &tmR, &k_full[st], 0, 0, row);
        }
        // a single stage of V is free once the product before has retired
        if (VS == 1 && j >= 1 && !mbar_wait(&kv_empty[(j - 1) & 1], ((j - 1) >> 1) & 1, p.err, ERR_ATTN_WAIT)) break;
        const int vs = j % VS;
        mbar_expect_tx(&v_full[vs], VA * ATOM_BYTES);
        tma_load_3d(smem + S::V + vs * TILE_BYTES, &tmV, &v_full[vs], 0, kv_head, row);
        if constexpr (VA > 1) tma_load_3d(smem + S::V + vs * TILE_BYTES + ATOM_BYTES, &tmV, &v_full[vs], 64, kv_head, row);
      }
    }
  } else if (warp == 9) {
    // ----------------------------------------------------------- MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(BQ, BKV, false, false);
      constexpr uint32_t idesc_o = umma_idesc_bf16(BQ, VA * 64, false, true);
      const uint32_t sq = smem_u32(smem + S::Q), sp = smem_u32(smem + S::P);
      auto issue_s = [&](int j) {
        const uint32_t sk = smem_u32(smem + S::K + (j & 1) * S::K_TILE);
#pragma unroll
        for (int k = 0; k < KA * 4; ++k) {
          const uint32_t off = (k >> 2) * ATOM_BYTES + (k & 3) * 32;
          umma_bf16(tmem_base + (j & 1) * 128, umma_desc(sq + off, 16, 1024), umma_desc(sk + off, 16, 1024), idesc_s, k ? 1u : 0u);
        }
        umma_commit(&s_full[j & 1]);
      };
      bool ok = mbar_wait(q_full, 0, p.err, ERR_ATTN_WAIT) && mbar_wait(&k_full[0], 0, p.err, ERR_ATTN_WAIT);
      if (ok) {
        tc_fence_after();
        issue_s(0);
      }
      for (int j = 0; ok && j < n_blocks; ++j) {
        if (j + 1 < n_blocks) {
          const int n = j + 1;
          ok = mbar_wait(&k_full[n & 1], (n >> 1) & 1, p.err, ERR_ATTN_WAIT);
          if (ok && n >= 2) ok = mbar_wait(&s_empty[n & 1], ((n >> 1) - 1) & 1, p.err, ERR_ATTN_WAIT);
          if (!ok) break;
          tc_fence_after();
          issue_s(n);
        }
        ok = mbar_wait(p_ready, j & 1, p.err, ERR_ATTN_WAIT) && mbar_wait(&v_full[j % VS], (j / VS) & 1, p.err, ERR_ATTN_WAIT);
        if (!ok) break;
        tc_fence_after();
        const uint32_t sv = smem_u32(smem + S::V + (j % VS) * TILE_BYTES);
#pragma unroll
        for (int k = 0; k < BKV / 16; ++k) {
          // A = P (K-major over kv): atom k/4, 32-byte step inside; B = V (MN-major): 16 kv rows = 2048 B per step
          const uint64_t ad = umma_desc(sp + (k >> 2) * ATOM_BYTES + (k & 3) * 32, 16, 1024);
          const uint64_t bd = umma_desc(sv + k * 2048, ATOM_BYTES, 1024);
          umma_bf16(tmem_o, ad, bd, idesc_o, (j > 0 || k > 0) ? 1u : 0u);
        }
        umma_commit(o_done);
        umma_commit(&kv_empty[j & 1]);
      }
    }
  } else {
    // -------------------------------------------------------------- softmax
    // Thread = (query row, half of the 128 key columns).  The 64 scores of its half stay in registers from the
    // max pass to the exp pass (one TMEM read per block); the two halves of a row agree on the row maximum
    // through shared memory + one named barrier per block.  A thread whose wait failed keeps taking part in the
    // barriers (doing no work) so that no thread is ever left waiting at one.
    const int wg = warp >> 2;
    const int row = (warp & 3) * 32 + lane;          // row inside the tile == TMEM lane
    const uint32_t lane_off = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const int q_pos = q0 + row;                      // position inside the sequence
    float* xmax = reinterpret_cast<float*>(smem + S::XCHG);   // [parity][half][128]
    float* xsum = xmax + 4 * 128;                                 // [half][128]
    // a row past the sequence's end keeps the bound of its place: what it computes is not stored
    const int first = bounded ? first_visible(max(q_pos + q_off, 0), p.window, p.chunk) : 0;
    const int first_last = bounded ? first_visible(max(q0 + BQ - 1 + q_off, 0), p.window, p.chunk) : 0;
    float m_used = -INFINITY, l_sum = 0.f;
    bool dead = false;
    // TERMS: band[j & 1][i] is the number for distance i − 127 between the tile's first query and key, in log2 units
    float* band = reinterpret_cast<float*>(smem + S::BAND);
    const DistanceNumber<bf16> number(p.terms, TERMS ? head : 0);
    const float score_scale = TERMS ? p.scale_log2 * 0.6931471805599453f * score_temp<bf16>(p.terms, head) : p.scale_log2;
    auto fill_band = [&](int j) {
      const int i = wg * 128 + row;
      band[(j & 1) * 256 + i] = number.at(max(q0 + q_off - (jb0 + j) * BKV + i - 127, 0)) * 1.4426950408889634f;
    };
    if constexpr (TERMS) {
      fill_band(0);
      asm volatile("bar.sync 1, 256;" ::: "memory");
    }
    for (int j = 0; j < n_blocks; ++j) {
      if (!dead && !mbar_wait(&s_full[j & 1], (j >> 1) & 1, p.err, ERR_ATTN_WAIT)) dead = true;
      const int kv0 = (jb0 + j) * BKV + wg * 64;
      float sc[64];
      float mx = -INFINITY;
      if (!dead) {
        tc_fence_after();
        const uint32_t ts = tmem_base + (j & 1) * 128 + wg * 64 + lane_off;
        uint32_t r0[32], r1[32];
        tmem_ld32(ts, r0);
        tmem_ld32(ts + 32, r1);
        tmem_ld_wait();
        tc_fence_before();
        mbar_arrive(&s_empty[j & 1]);                 // scores are in registers: the TMEM buffer may be refilled
        const bool need_mask = (kv0 + 64 > kv_end) || (p.causal && kv0 + 64 > q0 + q_off) || kv0 < first_last;
        if constexpr (TERMS) {
          if (p.terms.cap > 0.f) {
            const float to_u = score_scale * p.terms.inv_cap, cap_log2 = p.terms.cap * 1.4426950408889634f;
            float top = 0.f;
#pragma unroll
            for (int i = 0; i < 64; ++i) {
              sc[i] = __uint_as_float(i < 32 ? r0[i] : r1[i - 32]) * to_u;
              top = fmaxf(top, fabsf(sc[i]));
            }
            if (__any_sync(0xffffffffu, !(top <= kTanhNear))) {
#pragma unroll
              for (int i = 0; i < 64; ++i) sc[i] = cap_log2 * tanh_any(sc[i]);
            } else {           // the usual case: scores well inside the cap
#pragma unroll
              for (int i = 0; i < 64; ++i) sc[i] = cap_log2 * tanh_near(sc[i]);
            }
          } else {
#pragma unroll
            for (int i = 0; i < 64; ++i) sc[i] = __uint_as_float(i < 32 ? r0[i] : r1[i - 32]) * (score_scale * 1.4426950408889634f);
          }
          const float* mine = band + (j & 1) * 256 + row + 127 - wg * 64;
#pragma unroll
          for (int i = 0; i < 64; ++i) sc[i] += mine[-i];
        }
#pragma unroll
        for (int i = 0; i < 64; ++i) {
          float sv = TERMS ? sc[i] : __uint_as_float(i < 32 ? r0[i] : r1[i - 32]) * p.scale_log2;
          if (need_mask) {
            const int col = kv0 + i;
            if (col >= kv_end || col < first || (p.causal && col > q_pos + q_off)) sv = -INFINITY;
          }
          sc[i] = sv;
          mx = fmaxf(mx, sv);
        }
      }
      if constexpr (TERMS) fill_band(j + 1);
      xmax[((j & 1) * 2 + wg) * 128 + row] = mx;
      asm volatile("bar.sync 1, 256;" ::: "memory");
      mx = fmaxf(mx, xmax[((j & 1) * 2 + (wg ^ 1)) * 128 + row]);
      float alpha = 1.f;
      bool rescale = false;
      // a row may see none of its first blocks: its maximum then stays at −∞ and its weights are zero
      if (mx > m_used + RESCALE_THRESHOLD || (m_used == -INFINITY && mx != -INFINITY)) {
        alpha = (m_used == -INFINITY) ? 0.f : exp2f(m_used - mx);
        rescale = (j > 0);
        m_used = mx;
        l_sum *= alpha;
      }
      const float m_sub = m_used == -INFINITY ? 0.f : m_used;
      // P buffer and O accumulator are free once the previous P·V has retired
      if (!dead && j > 0 && !mbar_wait(o_done, (j - 1) & 1, p.err, ERR_ATTN_WAIT)) dead = true;
      if (dead) continue;
      tc_fence_after();
      if (wg < VA && __any_sync(0xffffffffu, rescale)) {
#pragma unroll 1
        for (int c = 0; c < 2; ++c) {
          uint32_t r[32];
          tmem_ld32(tmem_o + lane_off + wg * 64 + c * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
          tmem_st32(tmem_o + lane_off + wg * 64 + c * 32, r);
        }
        tmem_st_wait();
      }
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t packed[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float p0 = fast_exp2(sc[c * 32 + i] - m_sub), p1 = fast_exp2(sc[c * 32 + i + 1] - m_sub);
          // the sum uses the bf16-rounded values so that numerator and denominator match
          const __nv_bfloat162 pb = __floats2bfloat162_rn(p0, p1);
          l_sum += __low2float(pb) + __high2float(pb);
          packed[i >> 1] = *reinterpret_cast<const uint32_t*>(&pb);
        }
        store_row_chunk_sw128(smem + S::P, 128, row, wg * 64 + c * 32, packed);
      }
      tc_fence_before();
      fence_proxy_async();
      mbar_arrive(p_ready);
    }
    // ------------------------------------------------------------- epilogue
    xsum[wg * 128 + row] = l_sum;
    asm volatile("bar.sync 1, 256;" ::: "memory");
    l_sum += xsum[(wg ^ 1) * 128 + row];
    if (!dead && n_blocks > 0 && mbar_wait(o_done, (n_blocks - 1) & 1, p.err, ERR_ATTN_WAIT)) {
      tc_fence_after();
      if (p.sinks != nullptr) l_sum += exp2f(__bfloat162float(p.sinks[head]) * 1.4426950408889634f - m_used);
      float inv_l = (l_sum > 0.f) ? 1.f / l_sum : 0.f;
      const bool valid = q_pos < seq_len;
      const bf16* gate = p.gate.p != nullptr && valid ? reinterpret_cast<const bf16*>(p.gate.p) + static_cast<size_t>(seq_start + q_pos) * p.gate.ld + static_cast<size_t>(head) * max(p.gate.e, 1)
                                                      : nullptr;
      if (gate != nullptr && p.gate.e == 0) inv_l *= sigmoid_of(__bfloat162float(*gate));
      bf16* orow = p.out + (static_cast<size_t>(seq_start + q_pos) * p.hq + head) * p.e;
#pragma unroll 1
      for (int c = 2 * wg; c < 2 * wg + 2 && c * 32 < p.e; ++c) {
        uint32_t r[32];
        tmem_ld32(tmem_o + lane_off + c * 32, r);
        tmem_ld_wait();
        if (valid) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (VA == 1 || c >= 2) { if (c * 32 + i >= p.e) break; }
            if (gate != nullptr && p.gate.e > 0) {
              if (p.gate_vec) {
                const uint4 g = *reinterpret_cast<const uint4*>(gate + c * 32 + i);
                const uint32_t gw[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                  const float2 z = unpack_bf16(gw[x]);
                  r[i + 2 * x] = __float_as_uint(__uint_as_float(r[i + 2 * x]) * sigmoid_of(z.x));
                  r[i + 2 * x + 1] = __float_as_uint(__uint_as_float(r[i + 2 * x + 1]) * sigmoid_of(z.y));
                }
              } else {
#pragma unroll
                for (int x = 0; x < 8; ++x)
                  if (c * 32 + i + x < p.gate.e) r[i + x] = __float_as_uint(__uint_as_float(r[i + x]) * sigmoid_of(__bfloat162float(gate[c * 32 + i + x])));
              }
            }
            uint4 v = make_uint4(pack_bf16(__uint_as_float(r[i]) * inv_l, __uint_as_float(r[i + 1]) * inv_l),
                                 pack_bf16(__uint_as_float(r[i + 2]) * inv_l, __uint_as_float(r[i + 3]) * inv_l),
                                 pack_bf16(__uint_as_float(r[i + 4]) * inv_l, __uint_as_float(r[i + 5]) * inv_l),
                                 pack_bf16(__uint_as_float(r[i + 6]) * inv_l, __uint_as_float(r[i + 7]) * inv_l));
            *reinterpret_cast<uint4*>(orow + c * 32 + i) = v;
          }
        }
      }
      if (valid && wg == 0) p.lse[static_cast<size_t>(head) * p.T + seq_start + q_pos] = (m_used + log2f(l_sum)) * 0.6931471805599453f;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

// dims {D, H, T}: a box {64, 1, 128} is a [128 tokens][64] K-major swizzle atom of one head.
CUtensorMap make_head_tmap(const torch::Tensor& t, int rows) {
  return make_tmap_3d(t.data_ptr(), t.size(2), t.size(1), t.size(0), t.stride(1), t.stride(0), 64, 1, rows);
}

std::vector<torch::Tensor> flash_attn_fwd(const torch::Tensor& q, const torch::Tensor& k, const torch::Tensor& v, const torch::Tensor& cu,
                                          int64_t max_seqlen, bool causal, double scale, const c10::optional<torch::Tensor>& cu_k,
                                          const c10::optional<torch::Tensor>& sinks, const c10::optional<torch::Tensor>& gate, int64_t window, int64_t chunk,
                                          const c10::optional<torch::Tensor>& key_tail, double cap, const c10::optional<torch::Tensor>& temp, const c10::optional<torch::Tensor>& slope, const c10::optional<torch::Tensor>& rate, const c10::optional<torch::Tensor>& table, const c10::optional<torch::Tensor>& bucket) {
  TORCH_CHECK(q.is_cuda() && q.scalar_type() == torch::kBFloat16 && q.dim() == 3 && k.dim() == 3 && v.dim() == 3 && k.size(0) == v.size(0) && k.size(1) == v.size(1) &&
                  k.scalar_type() == torch::kBFloat16 && v.scalar_type() == torch::kBFloat16, "q [T,Hq,D], k [T,Hkv,D], v [T,Hkv,E] bf16");
  for (const auto* t : {&q, &k, &v})
    TORCH_CHECK(t->stride(2) == 1 && t->stride(1) % 8 == 0 && t->stride(0) % 8 == 0 && reinterpret_cast<uintptr_t>(t->data_ptr()) % 16 == 0,
                "q, k, v: unit stride inside a head, rows and heads on 16-byte boundaries");
  const bool tail = key_tail.has_value() && key_tail->defined();
  if (tail)
    TORCH_CHECK(key_tail->is_cuda() && key_tail->scalar_type() == torch::kBFloat16 && key_tail->dim() == 2 && key_tail->size(0) == k.size(0) && key_tail->size(1) % 8 == 0 &&
                    key_tail->size(1) > 0 && key_tail->size(1) <= 64 && key_tail->stride(1) == 1 && key_tail->stride(0) % 8 == 0 &&
                    reinterpret_cast<uintptr_t>(key_tail->data_ptr()) % 16 == 0, "shared key part [T, up to 64] bf16 on 16-byte boundaries");
  const int own_chunks = (static_cast<int>(k.size(2)) + 63) / 64, chunks = own_chunks + (tail ? 1 : 0);
  TORCH_CHECK(q.size(2) == k.size(2) + (tail ? key_tail->size(1) : 0) && k.size(2) % 8 == 0 && v.size(2) % 8 == 0 && k.size(2) > 0 && v.size(2) > 0 && chunks <= 3 && v.size(2) <= 128,
              "head widths: multiples of 8, keys up to 192 (three chunks of 64 with the shared part in one of its own), values up to 128");
  TORCH_CHECK(window >= 0 && chunk >= 0 && window < (int64_t(1) << 30) && chunk < (int64_t(1) << 30), "window and chunk: 0 (none) or positive");
  TORCH_CHECK(causal || (window == 0 && chunk == 0), "windows and chunks bound causal attention");
  TORCH_CHECK(cu.is_cuda() && cu.scalar_type() == torch::kInt32 && cu.is_contiguous(), "cu_seqlens int32 on device");
  TORCH_CHECK(q.size(1) % k.size(1) == 0, "Hq must be a multiple of Hkv");
  c10::cuda::CUDAGuard guard(q.device());
  const int T = q.size(0), hq = q.size(1), hkv = k.size(1), nseq = cu.numel() - 1;
  auto out = torch::empty({T, hq, v.size(2)}, q.options());
  auto lse = torch::empty({hq, T}, q.options().dtype(torch::kFloat32));
  if (T == 0 || nseq <= 0) return {out, lse};
  CUtensorMap tq = make_head_tmap(q, 128), tk_ = make_head_tmap(k, 128), tv = make_head_tmap(v, 128);
  CUtensorMap tr = tail ? make_tmap_3d(key_tail->data_ptr(), key_tail->size(1), 1, key_tail->size(0), key_tail->stride(0), key_tail->stride(0), 64, 1, 128) : tk_;
  FwdParams p{};
  p.out = reinterpret_cast<bf16*>(out.data_ptr()); p.lse = lse.data_ptr<float>(); p.e = v.size(2); p.cu = cu.data_ptr<int>();
  p.cu_k = p.cu;
  if (cu_k.has_value() && cu_k->defined()) {
    TORCH_CHECK(cu_k->is_cuda() && cu_k->scalar_type() == torch::kInt32 && cu_k->is_contiguous() && cu_k->numel() == cu.numel(), "cu_k like cu");
    p.cu_k = cu_k->data_ptr<int>();
  }
  if (sinks.has_value() && sinks->defined()) {
    TORCH_CHECK(sinks->is_cuda() && sinks->scalar_type() == torch::kBFloat16 && sinks->is_contiguous() && sinks->numel() == hq, "sinks [Hq] bf16");
    p.sinks = reinterpret_cast<const bf16*>(sinks->data_ptr());
  }
  p.gate = out_gate(gate, T, hq, v.size(2), torch::kBFloat16);
  p.gate_vec = p.gate.e == v.size(2) && p.gate.ld % 8 == 0 && reinterpret_cast<uintptr_t>(p.gate.p) % 16 == 0;
  p.terms = score_terms(cap, temp, slope, rate, table, bucket, hq, torch::kBFloat16);
  p.T = T; p.hq = hq; p.hkv = hkv; p.scale_log2 = static_cast<float>(scale * 1.4426950408889634); p.causal = causal; p.err = error_word();
  p.window = window; p.chunk = chunk; p.own_chunks = own_chunks; p.tail_col = k.size(2);
  const dim3 grid(hq, (static_cast<int>(max_seqlen) + fa::BQ - 1) / fa::BQ, nseq);
  auto stream = at::cuda::getCurrentCUDAStream();
#define TK_FLASH(KA, VA) do { if (p.terms.used) TK_FLASH_RUN(KA, VA, true); else TK_FLASH_RUN(KA, VA, false); } while (0)
#define TK_FLASH_RUN(KA, VA, TERMS)                                                                                                     \
  do {                                                                                                                                  \
    static bool configured = false;                                                                                                     \
    if (!configured) {                                                                                                                  \
      TK_CUDA_CHECK(cudaFuncSetAttribute(flash_fwd_kernel<KA, VA, TERMS>, cudaFuncAttributeMaxDynamicSharedMemorySize, fa::Smem<KA>::TOTAL));  \
      configured = true;                                                                                                                \
    }                                                                                                                                   \
    flash_fwd_kernel<KA, VA, TERMS><<<grid, fa::THREADS, fa::Smem<KA>::TOTAL, stream>>>(tq, tk_, tv, tr, p);                                   \
  } while (0)
  const bool wide_k = chunks > 1, wide_v = v.size(2) > 64;
  if (chunks == 3 && wide_v) TK_FLASH(3, 2);
  else if (chunks == 3) TK_FLASH(3, 1);
  else if (wide_k && wide_v) TK_FLASH(2, 2);
  else if (wide_k) TK_FLASH(2, 1);
  else if (wide_v) TK_FLASH(1, 2);
  else TK_FLASH(1, 1);
#undef TK_FLASH
#undef TK_FLASH_RUN
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return {out, lse};
}

}  // namespace tk
