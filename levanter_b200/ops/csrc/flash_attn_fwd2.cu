// Flash attention forward, two query tiles per CTA (sequence length a multiple of 256, head_dim 128).
//
// Compared with the one-tile kernel in flash_attn.cu this variant
//   * keeps two 128-row query tiles A and B per CTA, so every K/V tile fetched by TMA is used twice and
//     eight softmax warps (two per scheduler) hide each other's instruction latency;
//   * writes P back into the TMEM columns of S (bf16, two values per 32-bit column) and issues the
//     P V product with the A operand read from tensor memory, so P never touches shared memory;
//   * ping-pongs the tiles on the tensor core: while tile A's rows are in softmax the MMA warp runs
//     P_B V and Q_B K^T, and vice versa.
// TMEM map (512 columns): S_A/P_A [0,128)  S_B/P_B [128,256)  O_A [256,384)  O_B [384,512).
// Shared memory: Q_A, Q_B, two K stages, two V stages (6 x 32 KB).
// Mask semantics, outputs and the lazy-rescale rule are those of flash_fwd_kernel.
//
// kPacked (lvb_flash_attn_fwd_packed) is the form the inference engine prefills with: packed sequences, each starting at
// position 0.  What a row sees is one contiguous range of packed keys, so the mask is a lower bound per row computed from its
// position (the start of its sequence, of its chunk when attention is chunked, or of its window) instead of a segment id per
// key: blocks between the bound and the diagonal need no mask at all.  Key and value sizes may differ and need not be 64 or
// 128: the tensor maps are three-dimensional (size, head, row), columns past the size arrive as zeros, and the MMAs stop at
// the next multiple of 16.  Keys of up to 192 leave shared memory for one V stage only.  An optional gate is applied to the
// output on its way out.
//
// kMaps (kPacked only): differential attention.  The two tiles of a CTA are the two score maps of a head over the same 128 rows: each
// has queries and keys of its own (the K ring holds single tiles, alternating between the maps), both multiply the same V tile, and the
// epilogue forms a1 - weight * a2, its norm over the values and the gate straight from the two accumulators.  The warps of a tile
// take alternate groups of 32 columns of the result.
#include "common.cuh"

namespace lvb {
namespace fa2 {

constexpr int BT = 128;            // rows per query tile, keys per block
constexpr int kThreads = 320;      // warp0 TMA, warp1 MMA, warps 2-5 tile A, warps 6-9 tile B
constexpr int kTileBytes = 128 * 128 * 2;
constexpr int kChunkBytes = 128 * 64 * 2;
constexpr int kStages = 2;
constexpr float kRescaleThreshold = 8.0f;
constexpr float kLog2e = 1.4426950408889634f;

struct Params {
  __nv_bfloat16* O;
  float* lse2;
  const int* q_seg;
  const int* k_seg;
  const int* kblock_lo;  // optional [B, S / 128]: first block of 128 keys that a query of this 128-row block can attend to
  const float* sink;     // optional [Hq]: a learned logit per head that takes part in the softmax denominator only
  int B, S, Hq, Hkv;  // S: query positions per sequence
  int Sk;             // key positions per sequence (= S unless the mask has no causal part: cross attention)
  float scale, soft_cap;
  int window;
  int causal;  // 0: every key is visible (subject to segment ids); window must be 0 and kblock_lo null then
  int* status;
  // ---- kPacked
  const int* pos;            // [S]: position of each packed row in its sequence
  int chunk;                 // > 0: a row at position i sees positions >= i - i % chunk only (window, above: positions > i - window)
  int dk, dv;                // query/key and value sizes (multiples of 8, at most HD)
  const __nv_bfloat16* gate; // optional [S, Hq * dv], or [S, Hq] with gate_per_head (row stride ldg): the output is multiplied by its sigmoid
  long long ldg;
  int gate_per_head;
  // ---- kMaps: o = a1 - weight a2, then diff_scale * o / sqrt(mean(o^2) + eps)
  const float* weight;
  float diff_scale, eps;
};

// HDK, HDV: room for the query/key and the value size
template <int HDK, int HDV, bool kMaps = false>
struct SmemT {
  static constexpr int kQKTile = 128 * HDK * 2;               // a [128 rows, HDK] tile: HDK / 64 chunks of 64 columns
  static constexpr int kVTile = 128 * HDV * 2;
  static constexpr int kKStages = kMaps ? 2 * kStages : kStages;
  static constexpr int kVStages = HDK > (kMaps ? 64 : 128) ? 1 : kStages;
  static constexpr int kQ = 0;                                // 2 tiles
  static constexpr int kK = kQ + 2 * kQKTile;
  static constexpr int kV = kK + kKStages * kQKTile;
  static constexpr int kBars = kV + kVStages * kVTile;
  static constexpr int kNumBars = 1 + 2 * kKStages + 2 * kStages + 2 + 2 + 2;
  static constexpr int kTotal = kBars + kNumBars * 8 + 16 + 1024;
};

template <bool kValue>
struct Yes {  // a compile-time answer as an argument
  static constexpr bool value = kValue;
};

template <bool kCap>
__device__ __forceinline__ float to_log2(float s, float scale_log2, float scale, float cap) {
  // cap * tanh(s * scale / cap), from an exponential: this file's tanhf keeps about 11 bits
  if constexpr (kCap) return cap * kLog2e - __fdividef(2.f * kLog2e * cap, 1.f + exp2f(s * __fdividef(2.f * kLog2e * scale, cap)));
  else return s * scale_log2;
}

// kPacked: first packed key that row qi sees
__device__ __forceinline__ int row_lower_bound(const Params& p, int qi) {
  const int pos = p.pos[qi];
  const int back = p.chunk > 0 ? pos % p.chunk : pos;
  return qi - (p.window > 0 ? min(back, p.window - 1) : back);
}

// dst[0 .. 7] = f * e (times the sigmoid of gate[0 .. 7] when given)
__device__ __forceinline__ void store_row_piece(__nv_bfloat16* dst, const float* e, float f, const __nv_bfloat16* gate) {
  float v[8];
#pragma unroll
  for (int t = 0; t < 8; ++t) v[t] = e[t] * f;
  if (gate != nullptr) {
    const uint4 gw = __ldg(reinterpret_cast<const uint4*>(gate));
    const __nv_bfloat162* gh = reinterpret_cast<const __nv_bfloat162*>(&gw);
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      const float2 g = __bfloat1622float2(gh[t]);
      v[2 * t] *= 1.f / (1.f + __expf(-g.x));
      v[2 * t + 1] *= 1.f / (1.f + __expf(-g.y));
    }
  }
  *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
}

template <int HDK, int HDV, bool kSeg, bool kCap, bool kPacked = false, bool kMaps = false>
__global__ void __launch_bounds__(kThreads, 1)
flash_fwd2_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                  const __grid_constant__ CUtensorMap tmV, Params p) {
  static_assert(kPacked || !kMaps, "maps need packed rows");
  using Smem = SmemT<HDK, HDV, kMaps>;
  constexpr int kQKTile = Smem::kQKTile, kVTile = Smem::kVTile, kKStages = Smem::kKStages, kVStages = Smem::kVStages;
  constexpr int kRows = kMaps ? BT : 2 * BT;  // query rows per CTA
  const bool causal = p.causal != 0;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + Smem::kBars);
  uint64_t* q_full = bars;
  uint64_t* k_full = q_full + 1;
  uint64_t* k_empty = k_full + kKStages;
  uint64_t* v_full = k_empty + kKStages;
  uint64_t* v_empty = v_full + kStages;
  uint64_t* s_full = v_empty + kStages;  // [2 tiles]
  uint64_t* p_full = s_full + 2;         // [2 tiles]
  uint64_t* o_done = p_full + 2;         // [2 tiles]
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(o_done + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);

  const int warp = threadIdx.x >> 5;
  const int lane = threadIdx.x & 31;
  const int ncta = p.S / kRows;
  const int cb = ncta - 1 - static_cast<int>(blockIdx.x);  // heaviest first
  const int b = blockIdx.y / p.Hq;
  const int h = blockIdx.y % p.Hq;
  const int hkv = h / (p.Hq / p.Hkv);
  const int q0 = cb * kRows;
  // without the causal part there is no diagonal block (the mask test below never matches -1) and both tiles see every block
  const int jdiagA = kMaps ? cb : causal ? 2 * cb : -1, jdiagB = kMaps ? cb : causal ? 2 * cb + 1 : -1;
  int jlo = 0;
  if (!kPacked && p.window > 0) {
    const int first_key = q0 - p.window + 1;
    jlo = first_key > 0 ? first_key / BT : 0;
  }
  if (p.kblock_lo != nullptr) {
    // packed sequences (segment ids ascending): key blocks before the first query's sequence hold nothing these rows can see
    const int lo = p.kblock_lo[b * (p.S / BT) + jdiagA];
    jlo = max(jlo, min(lo, jdiagA));
  }
  if constexpr (kPacked) jlo = row_lower_bound(p, q0) / BT;  // bounds do not decrease along the packed rows
  const int nB = (causal ? jdiagB : p.Sk / BT - 1) - jlo + 1;  // blocks processed by tile B
  const int nA = causal && !kMaps ? nB - 1 : nB;              // causal: tile A stops one block earlier (its diagonal)

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    mbar_init(q_full, 1);
    for (int s = 0; s < kKStages; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
    }
    for (int s = 0; s < kStages; ++s) {
      mbar_init(&v_full[s], 1);
      mbar_init(&v_empty[s], 1);
    }
    for (int t = 0; t < 2; ++t) {
      mbar_init(&s_full[t], 1);
      mbar_init(&p_full[t], 4);
      mbar_init(&o_done[t], 1);
    }
    mbar_fence_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc<512>(tmem_holder);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_holder;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      const int row_q = b * p.S + q0;
      const int ck = kPacked ? (p.dk + 63) / 64 : HDK / 64, cv = kPacked ? (p.dv + 63) / 64 : HDV / 64;  // 64-column chunks
      mbar_expect_tx(q_full, 2 * ck * kChunkBytes);
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int c = 0; c < HDK / 64; ++c)
          if constexpr (kPacked) {
            if (c < ck) tma_load_3d(smem + Smem::kQ + t * kQKTile + c * kChunkBytes, &tmQ, q_full, 64 * c, kMaps ? 2 * h + t : h, kMaps ? row_q : row_q + t * BT);
          } else
          tma_load_2d(smem + Smem::kQ + t * kQKTile + c * kChunkBytes, &tmQ, q_full, h * HDK + 64 * c, row_q + t * BT);
      bool ok = true;
      for (int it = 0; it < nB && ok; ++it) {
        const int row_k = b * p.Sk + (jlo + it) * BT;
#pragma unroll
        for (int t = 0; t < (kMaps ? 2 : 1); ++t) {
          const int n = kMaps ? 2 * it + t : it, st = n % kKStages;
          ok = mbar_wait(&k_empty[st], ((n / kKStages) & 1) ^ 1, abort_flag, p.status, 1200, it);
          if (!ok) break;
          uint8_t* ks = smem + Smem::kK + st * kQKTile;
          mbar_expect_tx(&k_full[st], ck * kChunkBytes);
#pragma unroll
          for (int c = 0; c < HDK / 64; ++c)
            if constexpr (kPacked) {
              if (c < ck) tma_load_3d(ks + c * kChunkBytes, &tmK, &k_full[st], 64 * c, kMaps ? 2 * hkv + t : hkv, row_k);
            } else
            tma_load_2d(ks + c * kChunkBytes, &tmK, &k_full[st], hkv * HDK + 64 * c, row_k);
        }
        if (!ok) break;
        const int sv = it % kVStages;
        ok = mbar_wait(&v_empty[sv], ((it / kVStages) & 1) ^ 1, abort_flag, p.status, 1201, it);
        if (!ok) break;
        uint8_t* vs = smem + Smem::kV + sv * kVTile;
        mbar_expect_tx(&v_full[sv], cv * kChunkBytes);
#pragma unroll
        for (int c = 0; c < HDV / 64; ++c)
          if constexpr (kPacked) {
            if (c < cv) tma_load_3d(vs + c * kChunkBytes, &tmV, &v_full[sv], 64 * c, hkv, row_k);
          } else
          tma_load_2d(vs + c * kChunkBytes, &tmV, &v_full[sv], hkv * HDV + 64 * c, row_k);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_qk = make_idesc_bf16(BT, BT, false, false);
      // A = P in TMEM, B = V MN-major
      const uint32_t idesc_pv = make_idesc_bf16(BT, kPacked ? (p.dv + 15) / 16 * 16 : HDV, false, true);
      const int qk_steps = kPacked ? (p.dk + 15) / 16 : HDK / 16;
      const uint32_t sq = smem_u32(smem + Smem::kQ);
      bool ok = mbar_wait(q_full, 0, abort_flag, p.status, 1300, 0);

      auto k_tile = [&](int tile, int it) { return kMaps ? 2 * it + tile : it; };  // number of the K tile that a query tile meets
      auto qk = [&](int tile, int it) {
        const int st = k_tile(tile, it) % kKStages;
        const uint32_t sk = smem_u32(smem + Smem::kK + st * kQKTile);
        const uint32_t sqt = sq + tile * kQKTile;
#pragma unroll
        for (int kk = 0; kk < HDK / 16; ++kk) {
          if (kPacked && kk >= qk_steps) break;
          const uint32_t off = (kk >> 2) * kChunkBytes + (kk & 3) * 32;
          umma_bf16_ss(tmem_base + tile * BT, make_smem_desc(sqt + off, 16, 1024), make_smem_desc(sk + off, 16, 1024),
                       idesc_qk, kk > 0 ? 1u : 0u);
        }
        umma_commit(&s_full[tile]);
        if (kMaps || tile == 1) umma_commit(&k_empty[st]);
      };
      auto pv = [&](int tile, int it) {
        const uint32_t sv = smem_u32(smem + Smem::kV + (it % kVStages) * kVTile);
#pragma unroll
        for (int kk = 0; kk < BT / 16; ++kk) {
          // 16 keys of P = 8 TMEM columns; 16 keys of V = two 8-row groups = 2048 B
          umma_bf16_ts(tmem_base + 2 * BT + tile * HDV, tmem_base + tile * BT + kk * 8,
                       make_smem_desc(sv + kk * 2048, kChunkBytes, 1024), idesc_pv, (it > 0 || kk > 0) ? 1u : 0u);
        }
      };
      auto wait_k = [&](int tile, int it) {
        const int n = k_tile(tile, it);
        return mbar_wait(&k_full[n % kKStages], (n / kKStages) & 1, abort_flag, p.status, 1301, it);
      };
      auto wait_v = [&](int it) { return mbar_wait(&v_full[it % kVStages], (it / kVStages) & 1, abort_flag, p.status, 1302, it); };

      if (ok) ok = wait_k(0, 0);
      if (kMaps && ok) ok = wait_k(1, 0);
      if (ok) {
        tc_fence_after();
        qk(0, 0);
        qk(1, 0);
      }
      for (int it = 0; it < nB && ok; ++it) {
        ok = wait_v(it);
        if (!ok) break;
        if (it < nA) {
          ok = mbar_wait(&p_full[0], it & 1, abort_flag, p.status, 1303, it);
          if (!ok) break;
          tc_fence_after();
          pv(0, it);
          if (it == nA - 1) umma_commit(&o_done[0]);
        }
        const bool more = it + 1 < nB;
        if (more) {
          ok = wait_k(0, it + 1);
          if (!ok) break;
          tc_fence_after();
          if (it + 1 < nA) qk(0, it + 1);
        }
        ok = mbar_wait(&p_full[1], it & 1, abort_flag, p.status, 1304, it);
        if (!ok) break;
        tc_fence_after();
        pv(1, it);
        umma_commit(&v_empty[it % kVStages]);
        if (it == nB - 1) umma_commit(&o_done[1]);
        if (more) {
          if (kMaps) {
            ok = wait_k(1, it + 1);
            if (!ok) break;
            tc_fence_after();
          }
          qk(1, it + 1);
        }
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax + correction + epilogue
    const int tile = (warp - 2) >> 2;
    const int quad = warp & 3;
    const int r = quad * 32 + lane;
    const int tile_q0 = kMaps ? q0 : q0 + tile * BT;
    const int qi = tile_q0 + r;
    const int jdiag = tile == 0 ? jdiagA : jdiagB;
    const int nT = tile == 0 ? nA : nB;
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t tS = tmem_base + tile * BT + lane_addr;
    const uint32_t tO = tmem_base + 2 * BT + tile * HDV + lane_addr;
    const float scale_log2 = p.scale * kLog2e;
    const float cap_inv = kCap ? __fdividef(p.scale, p.soft_cap) : 0.f;
    const int my_seg = kSeg ? p.q_seg[b * p.S + qi] : 0;
    const int* kseg_row = kSeg ? p.k_seg + b * p.Sk : nullptr;
    float m_used = -INFINITY, l_sum = 0.f;
    bool ok = true;
    int row_lo = 0, tile_lo = 0;  // kPacked: this row's first visible key, and the last row's (the largest of the tile)
    if constexpr (kPacked) {
      row_lo = row_lower_bound(p, qi);
      tile_lo = row_lower_bound(p, tile_q0 + BT - 1);
    }

    for (int it = 0; it < nT && ok; ++it) {
      const int j = jlo + it;
      const int k0 = j * BT;
      ok = mbar_wait(&s_full[tile], it & 1, abort_flag, p.status, 1400 + tile, it);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const bool need_mask = (j == jdiag) || kSeg || (kPacked && k0 < tile_lo) || (!kPacked && p.window > 0 && k0 <= q0 + tile * BT + BT - 1 - p.window);

      // what the row sees of the block: columns col_lo .. col_lo + col_span (with segment ids: those of its segment)
      const int col_lo = (kPacked ? row_lo : p.window > 0 ? qi - p.window + 1 : 0) - k0;
      const unsigned col_span = causal ? static_cast<unsigned>(qi - k0 - col_lo) : 0x7fffffffu;
      uint32_t same[4] = {0u, 0u, 0u, 0u};  // kSeg: a bit per column, set in pass 1
      auto mask = [&](uint32_t (&v)[2][32], int c) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const uint32_t bits = c == 0 ? same[i] : same[2 + i];
#pragma unroll
          for (int t = 0; t < 32; ++t) {
            bool valid = static_cast<unsigned>(c + 32 * i + t - col_lo) <= col_span;
            if (kSeg) valid = valid && ((bits >> t) & 1u);
            if (!valid) v[i][t] = __float_as_uint(-INFINITY);
          }
        }
      };
      if constexpr (kSeg) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll 2
          for (int t = 0; t < 32; t += 4) {
            const int4 seg = __ldg(reinterpret_cast<const int4*>(kseg_row + k0 + 32 * i + t));
            same[i] |= (seg.x == my_seg ? 1u << t : 0u) | (seg.y == my_seg ? 2u << t : 0u) | (seg.z == my_seg ? 4u << t : 0u) |
                       (seg.w == my_seg ? 8u << t : 0u);
          }
      }

      // ---- pass 1: row maximum (raw logits; the scale is positive and the soft-cap monotonic).  Rolled loops over 64 columns: unrolled
      // further, the code no longer fits the instruction cache
      float mx0 = -INFINITY, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY, far0 = 0.f, far1 = 0.f;
#pragma unroll 1
      for (int c = 0; c < BT; c += 64) {
        uint32_t v[2][32];
        tmem_ld_32x32(tS + c, v[0]);
        tmem_ld_32x32(tS + c + 32, v[1]);
        tmem_ld_wait();
        if constexpr (kCap) {
#pragma unroll
          for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int t = 0; t < 32; t += 2) {
              far0 = fmaxf(far0, fabsf(__uint_as_float(v[i][t])));
              far1 = fmaxf(far1, fabsf(__uint_as_float(v[i][t + 1])));
            }
        }
        if (need_mask) mask(v, c);
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int t = 0; t < 32; t += 4) {
            mx0 = fmaxf(mx0, __uint_as_float(v[i][t]));
            mx1 = fmaxf(mx1, __uint_as_float(v[i][t + 1]));
            mx2 = fmaxf(mx2, __uint_as_float(v[i][t + 2]));
            mx3 = fmaxf(mx3, __uint_as_float(v[i][t + 3]));
          }
      }
      // kCap: whether all logits of the warp lie where the cap is a polynomial
      const bool near = kCap && __all_sync(0xffffffffu, fmaxf(far0, far1) * p.scale <= 0.75f * p.soft_cap);
      const float m_raw = fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3));
      const float m_blk = (m_raw == -INFINITY) ? -INFINITY : to_log2<kCap>(m_raw, scale_log2, p.scale, p.soft_cap);

      // ---- lazy rescale of O (S_T ready implies the previous P_T V has retired).  The decision is per row, but the
      // TMEM load/store are warp-collective, so the whole warp takes the branch as soon as one row needs it and rows
      // that do not need it scale by exactly 1.
      {
        const bool want = (m_blk > m_used + kRescaleThreshold) || (m_used == -INFINITY && m_blk > -INFINITY);
        const float m_new = want ? fmaxf(m_used, m_blk) : m_used;
        const bool scale_row = want && it > 0 && m_used > -INFINITY;
        if (__any_sync(0xffffffffu, scale_row)) {
          const float alpha = scale_row ? exp2f(m_used - m_new) : 1.f;
          l_sum *= alpha;
#pragma unroll 1
          for (int c = 0; c < HDV; c += 16) {  // few columns at a time: the logits hold most registers
            uint32_t w[16];
            tmem_ld_32x16(tO + c, w);
            tmem_ld_wait();
#pragma unroll
            for (int t = 0; t < 16; ++t) w[t] = __float_as_uint(__uint_as_float(w[t]) * alpha);
            tmem_st_32x16(tO + c, w);
          }
        }
        m_used = m_new;
      }
      const float neg_m = (m_used == -INFINITY) ? 0.f : -m_used;

      // ---- pass 2: P = exp2(s - m) -> bf16 pairs written over the first 64 columns of S
      const F32x2 scale2 = f2(scale_log2, scale_log2), cap2 = f2(cap_inv, cap_inv), neg2 = f2(neg_m, neg_m);
      F32x2 sum[4] = {f2(0.f, 0.f), f2(0.f, 0.f), f2(0.f, 0.f), f2(0.f, 0.f)};
      auto exponentials = [&](auto masked, auto polynomial) {
        constexpr bool kMasked = decltype(masked)::value, kPoly = decltype(polynomial)::value;
#pragma unroll 1
        for (int c = 0; c < BT; c += 64) {
          uint32_t v[2][32];
          tmem_ld_32x32(tS + c, v[0]);
          tmem_ld_32x32(tS + c + 32, v[1]);
          tmem_ld_wait();
          if constexpr (kMasked) mask(v, c);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            uint32_t pk[16];
#pragma unroll
            for (int t = 0; t < 16; ++t) {
              const float x0 = __uint_as_float(v[i][2 * t]), x1 = __uint_as_float(v[i][2 * t + 1]);
              const F32x2 x = f2(x0, x1);
              float a, b;
              if constexpr (!kCap) {
                f2_split(f2_fma(x, scale2, neg2), a, b);
              } else if constexpr (kPoly) {
                const F32x2 y = f2_mul(x, cap2);
                f2_split(f2_fma(f2_mul(x, scale2), tanh_ratio(f2_mul(y, y)), neg2), a, b);
              } else {
                a = to_log2<kCap>(x0, scale_log2, p.scale, p.soft_cap) + neg_m;
                b = to_log2<kCap>(x1, scale_log2, p.scale, p.soft_cap) + neg_m;
              }
              if constexpr (kCap && kMasked) {  // a masked logit does not stay masked under the cap
                a = x0 == -INFINITY ? -INFINITY : a;
                b = x1 == -INFINITY ? -INFINITY : b;
              }
              a = exp2f(a);
              b = exp2f(b);
              sum[t & 3] = f2_add(sum[t & 3], f2(a, b));
              pk[t] = pack_bf16x2(a, b);
            }
            tmem_st_32x16(tS + (c >> 1) + 16 * i, pk);
          }
        }
      };
      if (kCap && !near) exponentials(Yes<true>{}, Yes<false>{});
      else if (need_mask) exponentials(Yes<true>{}, Yes<true>{});
      else exponentials(Yes<false>{}, Yes<true>{});
      float s0, s1;
      f2_split(f2_add(f2_add(sum[0], sum[1]), f2_add(sum[2], sum[3])), s0, s1);
      l_sum += s0 + s1;
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[tile]);
    }

    if constexpr (kMaps) {
      // the queries are not needed any more: their memory carries the rows' sums and partial norms between the two tiles' warps
      for (int i = 0; i < 2 && ok; ++i) ok = mbar_wait(&o_done[i], 0, abort_flag, p.status, 1410 + i, nT);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      float* s_inv = reinterpret_cast<float*>(smem + Smem::kQ);  // [2][BT]
      float* s_ss = s_inv + 2 * BT;                              // [2][BT]
      if (ok) s_inv[tile * BT + r] = l_sum > 0.f ? 1.f / l_sum : 0.f;
      named_bar_sync(1, 8 * 32);
      const uint32_t tO1 = tmem_base + 2 * BT + lane_addr, tO2 = tO1 + HDV;
      constexpr int kGroups = HDV / 64;  // groups of 32 columns per warp
      float o[kGroups][32], ss = 0.f;
      const float c1 = s_inv[r], c2 = -*p.weight * s_inv[BT + r];
#pragma unroll
      for (int n = 0; n < kGroups; ++n) {
        const int c = (2 * n + tile) * 32;
        if (c < p.dv) {
          uint32_t v1[32], v2[32];
          tmem_ld_32x32(tO1 + c, v1);
          tmem_ld_32x32(tO2 + c, v2);
          tmem_ld_wait();
#pragma unroll
          for (int t = 0; t < 32; ++t) {
            o[n][t] = c + t < p.dv ? fmaf(c1, __uint_as_float(v1[t]), c2 * __uint_as_float(v2[t])) : 0.f;
            ss = fmaf(o[n][t], o[n][t], ss);
          }
        }
      }
      if (ok) s_ss[tile * BT + r] = ss;
      named_bar_sync(1, 8 * 32);
      if (ok) {
        float f = p.diff_scale * rsqrtf((s_ss[r] + s_ss[BT + r]) / static_cast<float>(p.dv) + p.eps);
        const __nv_bfloat16* grow = nullptr;
        if (p.gate != nullptr) {
          if (p.gate_per_head) f *= 1.f / (1.f + __expf(-__bfloat162float(p.gate[static_cast<size_t>(qi) * p.ldg + h])));
          else grow = p.gate + static_cast<size_t>(qi) * p.ldg + static_cast<size_t>(h) * p.dv;
        }
        __nv_bfloat16* orow = p.O + (static_cast<size_t>(qi) * p.Hq + h) * p.dv;
#pragma unroll
        for (int n = 0; n < kGroups; ++n) {
          const int c = (2 * n + tile) * 32;
#pragma unroll
          for (int q4 = 0; q4 < 4; ++q4)
            if (c + 8 * q4 < p.dv) store_row_piece(orow + c + 8 * q4, &o[n][8 * q4], f, grow != nullptr ? grow + c + 8 * q4 : nullptr);
        }
      }
    } else {
    if (ok) {
      ok = mbar_wait(&o_done[tile], 0, abort_flag, p.status, 1410 + tile, nT);
      ok = __all_sync(0xffffffffu, ok);
    }
    if (ok) {
      tc_fence_after();
      float o_scale = 1.f;
      if (p.sink != nullptr) {
        // The sink is one more column of the softmax whose value row is zero: it enters the denominator (and the saved
        // log-sum-exp) and nothing else.  If it raises the reference maximum from m to m', the accumulated output and sum
        // (both relative to m) shrink by a = 2^(m - m').
        const float s2 = p.sink[h] * kLog2e;
        const float m_new = fmaxf(m_used, s2);
        o_scale = (m_used == -INFINITY) ? 0.f : exp2f(m_used - m_new);
        l_sum = l_sum * o_scale + exp2f(s2 - m_new);
        m_used = m_new;
      }
      const float inv = l_sum > 0.f ? o_scale / l_sum : 0.f;
      if constexpr (kPacked) {
        __nv_bfloat16* orow = p.O + static_cast<size_t>(qi) * (static_cast<size_t>(p.Hq) * p.dv) + static_cast<size_t>(h) * p.dv;
        const __nv_bfloat16* grow = nullptr;
        float f = inv;
        if (p.gate != nullptr) {
          if (p.gate_per_head) f *= 1.f / (1.f + __expf(-__bfloat162float(p.gate[static_cast<size_t>(qi) * p.ldg + h])));
          else grow = p.gate + static_cast<size_t>(qi) * p.ldg + static_cast<size_t>(h) * p.dv;
        }
#pragma unroll 1
        for (int c = 0; c < p.dv; c += 32) {
          uint32_t v[32];
          tmem_ld_32x32(tO + c, v);
          tmem_ld_wait();
          float e[32];
#pragma unroll
          for (int t = 0; t < 32; ++t) e[t] = __uint_as_float(v[t]);
#pragma unroll
          for (int q4 = 0; q4 < 4; ++q4)
            if (c + 8 * q4 < p.dv) store_row_piece(orow + c + 8 * q4, e + 8 * q4, f, grow != nullptr ? grow + c + 8 * q4 : nullptr);
        }
      } else {
      __nv_bfloat16* orow = p.O + (static_cast<size_t>(b) * p.S + qi) * (static_cast<size_t>(p.Hq) * HDV) + static_cast<size_t>(h) * HDV;
#pragma unroll 1
      for (int c = 0; c < HDV; c += 32) {
        uint32_t v[32];
        tmem_ld_32x32(tO + c, v);
        tmem_ld_wait();
#pragma unroll
        for (int q4 = 0; q4 < 4; ++q4) {
          uint4 w;
          w.x = pack_bf16x2(__uint_as_float(v[q4 * 8 + 0]) * inv, __uint_as_float(v[q4 * 8 + 1]) * inv);
          w.y = pack_bf16x2(__uint_as_float(v[q4 * 8 + 2]) * inv, __uint_as_float(v[q4 * 8 + 3]) * inv);
          w.z = pack_bf16x2(__uint_as_float(v[q4 * 8 + 4]) * inv, __uint_as_float(v[q4 * 8 + 5]) * inv);
          w.w = pack_bf16x2(__uint_as_float(v[q4 * 8 + 6]) * inv, __uint_as_float(v[q4 * 8 + 7]) * inv);
          reinterpret_cast<uint4*>(orow + c)[q4] = w;
        }
      }
      p.lse2[(static_cast<size_t>(b) * p.Hq + h) * p.S + qi] = (l_sum > 0.f) ? m_used + log2f(l_sum) : -INFINITY;
      }
    }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc<512>(tmem_base);
  }
}

template <int HDK, int HDV, bool kSeg, bool kCap, bool kPacked = false, bool kMaps = false>
int launch(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV, const Params& p, cudaStream_t st) {
  using Smem = SmemT<HDK, HDV, kMaps>;
  static_assert(Smem::kTotal <= 227 * 1024, "shared memory of one CTA");
  auto kern = flash_fwd2_kernel<HDK, HDV, kSeg, kCap, kPacked, kMaps>;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Smem::kTotal) != cudaSuccess) return kErrCuda;
    attr_set = true;
  }
  dim3 grid(p.S / (kMaps ? BT : 2 * BT), p.B * p.Hq);
  kern<<<grid, kThreads, Smem::kTotal, st>>>(tmQ, tmK, tmV, p);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

}  // namespace fa2
}  // namespace lvb

namespace lvb {
namespace fa2 {
template <int HD>
int launch_hd(const void* q, const void* k, const void* v, const Params& p, cudaStream_t st) {
  CUtensorMap tmQ, tmK, tmV;
  const uint64_t rows = static_cast<uint64_t>(p.B) * p.S;
  int rc = make_tmap_2d_bf16(&tmQ, q, rows, static_cast<uint64_t>(p.Hq) * HD, static_cast<uint64_t>(p.Hq) * HD, BT, 64);
  if (rc != kErrOk) return rc;
  const uint64_t rows_k = static_cast<uint64_t>(p.B) * p.Sk;
  rc = make_tmap_2d_bf16(&tmK, k, rows_k, static_cast<uint64_t>(p.Hkv) * HD, static_cast<uint64_t>(p.Hkv) * HD, BT, 64);
  if (rc != kErrOk) return rc;
  rc = make_tmap_2d_bf16(&tmV, v, rows_k, static_cast<uint64_t>(p.Hkv) * HD, static_cast<uint64_t>(p.Hkv) * HD, BT, 64);
  if (rc != kErrOk) return rc;
  const bool seg = p.q_seg != nullptr;
  const bool cap = p.soft_cap > 0.f;
  if (seg && cap) return launch<HD, HD, true, true>(tmQ, tmK, tmV, p, st);
  if (seg) return launch<HD, HD, true, false>(tmQ, tmK, tmV, p, st);
  if (cap) return launch<HD, HD, false, true>(tmQ, tmK, tmV, p, st);
  return launch<HD, HD, false, false>(tmQ, tmK, tmV, p, st);
}
}  // namespace fa2
}  // namespace lvb

// Same contract as lvb_flash_attn_fwd_hd (head_dim 64 or 128, causal or not, optional sink logits [Hq]), but S must be a
// multiple of 256: two query tiles per CTA.  Sk: keys per sequence, a multiple of 128 (k / v are [B, Sk, Hkv, D], k_seg [B, Sk]);
// Sk must equal S when causal.
extern "C" int lvb_flash_attn_fwd2_hd(const void* q, const void* k, const void* v, void* o, float* lse2, const int* q_seg,
                                      const int* k_seg, const int* kblock_lo, const float* sink, int B, int S, int Sk, int Hq, int Hkv,
                                      int head_dim, int causal, float scale, float soft_cap, int window, int* status, void* stream) {
  using namespace lvb;
  using namespace lvb::fa2;
  if (B <= 0 || S <= 0 || (S % (2 * BT)) != 0 || Hq <= 0 || Hkv <= 0 || (Hq % Hkv) != 0) return kErrBadArg;
  if (!causal && (window != 0 || kblock_lo != nullptr)) return kErrBadArg;
  if (Sk <= 0 || (Sk % BT) != 0 || (causal && Sk != S)) return kErrBadArg;
  if (reinterpret_cast<uintptr_t>(k_seg) & 15) return kErrBadArg;
  Params p;
  p.O = reinterpret_cast<__nv_bfloat16*>(o);
  p.lse2 = lse2;
  p.q_seg = q_seg;
  p.k_seg = k_seg;
  p.kblock_lo = kblock_lo;
  p.sink = sink;
  p.B = B; p.S = S; p.Sk = Sk; p.Hq = Hq; p.Hkv = Hkv;
  p.scale = scale; p.soft_cap = soft_cap; p.window = window;
  p.causal = causal ? 1 : 0;
  p.status = status;
  p.pos = nullptr; p.chunk = 0; p.dk = p.dv = head_dim; p.gate = nullptr; p.ldg = 0; p.gate_per_head = 0;
  p.weight = nullptr; p.diff_scale = p.eps = 0.f;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (head_dim == 128) return launch_hd<128>(q, k, v, p, st);
  if (head_dim == 64) return launch_hd<64>(q, k, v, p, st);
  return kErrBadArg;
}

// Causal, head_dim 128 (the original entry point).
extern "C" int lvb_flash_attn_fwd2(const void* q, const void* k, const void* v, void* o, float* lse2, const int* q_seg,
                                   const int* k_seg, const int* kblock_lo, int B, int S, int Hq, int Hkv, float scale, float soft_cap,
                                   int window, int* status, void* stream) {
  return lvb_flash_attn_fwd2_hd(q, k, v, o, lse2, q_seg, k_seg, kblock_lo, nullptr, B, S, S, Hq, Hkv, 128, 1, scale, soft_cap, window, status, stream);
}

// Causal attention over T packed rows (T a multiple of 256) of sequences that each start at position 0:
//   q: row t, head h at q + t * ldq + h * dk     k / v: row t, head g at k + t * ldk + g * dk, v + t * ldv + g * dv
//   o[T, Hq, dv] = softmax(scale q k^T over the visible keys) v  (* sigmoid(gate[t, h, :]) or sigmoid(gate[t, h]) with gate_per_head)
// pos[t] is the row's position in its sequence (padding rows: 0).  chunk > 0: positions are cut into chunks of that many, counted
// from the sequence's start, and a row sees its own chunk only; window > 0: a row sees itself and the window - 1 positions before
// it.  sink (optional, fp32 [Hq]): joins the softmax denominator as it is.  weight (optional, one fp32 number on the device): q and k hold two
// score maps per head side by side (rows of 2 Hq and 2 Hkv heads), and o = diff_scale * d / sqrt(mean(d^2) + eps) with d = a1 - weight * a2
// (no sink then).  dk, dv: multiples of 8, at most 192 (128 with two maps) and 128; ldq, ldk, ldv and, for a gate per element, ldg
// multiples of 8 and the pointers 16-byte aligned.
extern "C" int lvb_flash_attn_fwd_packed(const void* q, const void* k, const void* v, const void* gate, const float* sink, void* o, const int* pos,
                                         int T, int Hq, int Hkv, int dk, int dv, int ldq, int ldk, int ldv, int ldg, int gate_per_head,
                                         int chunk, int window, float scale, float soft_cap, const float* weight, float diff_scale,
                                         float eps, int* status, void* stream) {
  using namespace lvb;
  using namespace lvb::fa2;
  if (T <= 0 || (T % (2 * BT)) != 0 || Hq <= 0 || Hkv <= 0 || (Hq % Hkv) != 0 || pos == nullptr || chunk < 0 || window < 0) return kErrBadArg;
  if (dk <= 0 || dv <= 0 || dk > (weight != nullptr ? 128 : 192) || dv > 128 || (dk & 7) || (dv & 7) || !(scale > 0.f)) return kErrBadArg;
  if (gate != nullptr && !gate_per_head && ((ldg & 7) || (reinterpret_cast<uintptr_t>(gate) & 15))) return kErrBadArg;
  if ((reinterpret_cast<uintptr_t>(o) & 15) || (weight != nullptr && sink != nullptr)) return kErrBadArg;
  Params p;
  p.O = reinterpret_cast<__nv_bfloat16*>(o);
  p.lse2 = nullptr; p.q_seg = nullptr; p.k_seg = nullptr; p.kblock_lo = nullptr; p.sink = sink;
  p.B = 1; p.S = T; p.Sk = T; p.Hq = Hq; p.Hkv = Hkv;
  p.scale = scale; p.soft_cap = soft_cap; p.window = window; p.causal = 1; p.status = status;
  p.pos = pos; p.chunk = chunk; p.dk = dk; p.dv = dv;
  p.gate = reinterpret_cast<const __nv_bfloat16*>(gate); p.ldg = ldg; p.gate_per_head = gate_per_head;
  p.weight = weight; p.diff_scale = diff_scale; p.eps = eps;
  const int maps = weight != nullptr ? 2 : 1;
  CUtensorMap tmQ, tmK, tmV;
  int rc = make_tmap_heads_bf16(&tmQ, q, T, Hq * maps, dk, ldq, BT);
  if (rc == kErrOk) rc = make_tmap_heads_bf16(&tmK, k, T, Hkv * maps, dk, ldk, BT);
  if (rc == kErrOk) rc = make_tmap_heads_bf16(&tmV, v, T, Hkv, dv, ldv, BT);
  if (rc != kErrOk) return rc;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const bool small = dk <= 64 && dv <= 64;
  if (maps == 2) {
    if (soft_cap > 0.f)
      return dk <= 64 ? launch<64, 128, false, true, true, true>(tmQ, tmK, tmV, p, st) : launch<128, 128, false, true, true, true>(tmQ, tmK, tmV, p, st);
    return dk <= 64 ? launch<64, 128, false, false, true, true>(tmQ, tmK, tmV, p, st) : launch<128, 128, false, false, true, true>(tmQ, tmK, tmV, p, st);
  }
  if (soft_cap > 0.f) {
    if (dk > 128) return launch<192, 128, false, true, true>(tmQ, tmK, tmV, p, st);
    return small ? launch<64, 64, false, true, true>(tmQ, tmK, tmV, p, st) : launch<128, 128, false, true, true>(tmQ, tmK, tmV, p, st);
  }
  if (dk > 128) return launch<192, 128, false, false, true>(tmQ, tmK, tmV, p, st);
  return small ? launch<64, 64, false, false, true>(tmQ, tmK, tmV, p, st) : launch<128, 128, false, false, true>(tmQ, tmK, tmV, p, st);
}
