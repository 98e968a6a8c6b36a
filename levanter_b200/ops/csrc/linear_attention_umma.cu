// The chunked form of linear attention with fixed decays (linear_attention.cu says what it computes) for keys of up to 128, on tcgen05.
//
// A work item is one piece of one head, for 64 columns of the values, walked in chunks of 128 rows; a persistent CTA per SM takes items in
// turn, and the copies of the next item start before the present one ends.  Per chunk, with the state S [dk, 64] as an fp32 accumulator
// in tensor memory:
//   A = Q K^T (128 x 128)        -> P = A o decays, bf16, in tensor memory again (row i, keys up to i; the rest stays zero)
//   O1 = Q [S_hi | S_lo]         S is written to shared memory in two bf16 parts, side by side, before the chunk touches it
//   O2 = P V,  out = decay^(i+1) (O1_hi + O1_lo) + O2
//   S <- decay^n S + K^T [V_hi | V_lo]   with the decayed values in two bf16 parts, and S the sum of its accumulator's halves
// Side by side the two parts are one MMA of 128 columns, which reads the other factor once.
//
// The chains from one chunk to the next are what takes time, so the roles meet as late as they can: warp 0 fetches Q, K and V by TMA two
// chunks deep; warp 1 issues A of a chunk and then O2 of the one before, warp 2 the products of the state; warps 4-7 make P of a chunk and
// then write the outputs of the one before, warps 8-11 carry the state, warps 12-15 decay the values.  Their loops are kept short on
// purpose: unrolled, the roles together do not fit the instruction cache, and everything takes twice as long.
// TMEM map (512 columns): A [0, 128)  P [128, 192)  O2 [192, 256)  O1 [256, 384)  S [384, 512).
#include "linear_attention.cuh"

namespace lvb {
namespace linattn {

constexpr int kUC = 128;             // rows of a chunk
constexpr int kUThreads = 512;
constexpr int kUTile = 128 * 64 * 2; // 128 rows of 64 columns

struct USmem {
  static constexpr int kQ = 0, kK = 2 * kUTile, kV = 4 * kUTile;  // within a stage
  static constexpr int kStage = 5 * kUTile;
  static constexpr int kState = 2 * kStage;            // S in two parts
  static constexpr int kValues = kState + 2 * kUTile;  // decayed V in two parts
  static constexpr int kPow = kValues + 2 * kUTile;    // key_scale * (32 zeros, decay^0 .. decay^127)
  static constexpr int kBars = kPow + 160 * 4;
  static constexpr int kNumBars = 12;
  static constexpr int kTotal = kBars + kNumBars * 8 + 16 + 1024;
};
static_assert(USmem::kTotal <= 227 * 1024, "shared memory of one CTA");

// A descriptor `bytes` further on.
__device__ __forceinline__ uint64_t ahead(uint64_t desc, uint32_t bytes) { return desc + (bytes >> 4); }

// One work item.
struct Item {
  int h, c0, seq, piece, of;  // columns c0 .. c0 + 63 of head h; piece number of the sequence and of how many
  int index;                  // of the piece among all pieces
  int r0, rows, chunks;
  Sequence s;
};

// kStateOnly: what a piece adds to a zero state, for all pieces but the last of a sequence.
template <bool kStateOnly>
__global__ void __launch_bounds__(kUThreads, 1)
umma_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long ldo = static_cast<long long>(p.H) * p.dv, head = static_cast<long long>(p.dk) * p.dv;
  const int slices = (p.dv + 63) / 64, per_piece = slices * p.H;
  const int ck = (p.dk + 63) / 64;  // 64-column parts of queries and keys

  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + USmem::kBars);
  uint64_t* full = bars;           // [2 stages] Q, K and V have arrived
  uint64_t* empty = bars + 2;      // [2 stages] and are not needed any more
  uint64_t* a_full = bars + 4;     // A is complete
  uint64_t* o1_full = bars + 5;    // O1 is complete: the state in shared memory has been read
  uint64_t* o2_full = bars + 6;    // O2 is complete: P has been read
  uint64_t* s_full = bars + 7;     // the state has taken up the chunk: the decayed values have been read
  uint64_t* p_full = bars + 8;     // P is in place, A has been read         (from here on four warps arrive)
  uint64_t* o_read = bars + 9;     // O1 and O2 have been read
  uint64_t* s_ready = bars + 10;   // the state is in shared memory, and decayed in its accumulator
  uint64_t* v_ready = bars + 11;   // the decayed values are in place
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bars + USmem::kNumBars);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);
  if (threadIdx.x == 0) {
    *abort_flag = 0;
    for (int i = 0; i < USmem::kNumBars; ++i) mbar_init(&bars[i], i >= 8 ? 4 : (i == 2 || i == 3) && !kStateOnly ? 2 : 1);
    mbar_fence_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc<512>(tmem_holder);
    tmem_relinquish();
  }
  if (ck == 1) {  // the upper rows of the state's tile multiply zeros
    for (int i = threadIdx.x; i < 2 * kUTile / 16; i += kUThreads) {
      const int st = i / (kUTile / 16), u = i % (kUTile / 16);
      *reinterpret_cast<uint4*>(smem + st * USmem::kStage + USmem::kK + kUTile + u * 16) = make_uint4(0u, 0u, 0u, 0u);
    }
    fence_proxy_async_smem();
  }
  if constexpr (!kStateOnly) {  // rows of no sequence come out as zeros
    const int n_seq = live_sequences(p);
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out);
    for (int r = (n_seq > 0 ? p.cu_q_lens[n_seq] : 0) + blockIdx.x; r < p.T; r += gridDim.x)
      for (long long e = threadIdx.x * 8; e < ldo; e += kUThreads * 8) *reinterpret_cast<uint4*>(out + r * ldo + e) = make_uint4(0u, 0u, 0u, 0u);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;
  const uint32_t tA = tmem, tP = tmem + 128, tO2 = tmem + 192, tO1 = tmem + 256, tS = tmem + 384;
  const int quad = warp & 3, row = quad * 32 + lane;
  const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;

  // The w-th work item.  0: there are no more, 1: nothing to do here, 2: there it is.  All lanes of a warp together.
  auto item_at = [&](int w, Item& it) {
    it.index = w / per_piece;
    it.h = w % per_piece / slices;
    it.c0 = w % slices * 64;
    if (!find_piece(p, it.index, it.seq, it.piece, it.of)) return 0;
    if (!sequence(p, it.seq, it.s) || (kStateOnly && it.piece == it.of - 1)) return 1;
    it.r0 = it.s.r0 + it.piece * p.piece;
    it.rows = min(p.piece, it.s.r1 - it.r0);
    it.chunks = (it.rows + kUC - 1) / kUC;
    return 2;
  };
  // for warps that go on to collective instructions: all lanes or none
  auto wait_all = [&](uint64_t* bar, uint32_t parity, int site, int extra) {
    return __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag, p.status, site, extra)) != 0;
  };
  auto arrive = [&](uint64_t* bar) {
    __syncwarp();
    if (lane == 0) mbar_arrive(bar);
  };
  Item it;
  int k = 0;  // chunks so far, of all items: what the parities count
  bool ok = true;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    for (int w = blockIdx.x, have; ok && (have = item_at(w, it)) != 0; w += gridDim.x) {
      if (have == 1) continue;
      if (lane == 0) {
        for (int c = 0; c < it.chunks; ++c) {
          const int n = k + c, st = n & 1;
          ok = mbar_wait(&empty[st], ((n >> 1) & 1) ^ 1, abort_flag, p.status, 1700, n);
          if (!ok) {  // let the copies in flight land
            for (int i = max(n - 2, 0); i < n; ++i) mbar_wait_quiet(&full[i & 1], (i >> 1) & 1);
            break;
          }
          uint8_t* at = smem + st * USmem::kStage;
          mbar_expect_tx(&full[st], ((kStateOnly ? 1 : 2) * ck + 1) * kUTile);
          const int r = it.r0 + c * kUC;
          for (int i = 0; i < ck; ++i) {
            if (!kStateOnly) tma_load_3d(at + USmem::kQ + i * kUTile, &tmQ, &full[st], 64 * i, it.h, r);
            tma_load_3d(at + USmem::kK + i * kUTile, &tmK, &full[st], 64 * i, it.h, r);
          }
          tma_load_3d(at + USmem::kV, &tmV, &full[st], it.c0, it.h, r);
        }
      }
      ok = __all_sync(0xffffffffu, ok) != 0;
      k += it.chunks;
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ A = Q K^T, and O2 = P V of the chunk before
    if constexpr (!kStateOnly) {
      constexpr uint32_t id_qk = make_idesc_bf16(128, 128, false, false);
      constexpr uint32_t id_pv = make_idesc_bf16(128, 64, false, true);  // V by rows of the inner index
      const int steps = (p.dk + 15) / 16;
      const uint32_t base = smem_u32(smem);
      const uint64_t d_q = make_smem_desc(base + USmem::kQ, 16, 1024), d_k = make_smem_desc(base + USmem::kK, 16, 1024);
      const uint64_t d_v = make_smem_desc(base + USmem::kV, kUTile, 1024);
      auto product_pv = [&](int n) {
        const uint64_t v = ahead(d_v, (n & 1) * USmem::kStage);
        ok = mbar_wait(o_read, (n & 1) ^ 1, abort_flag, p.status, 1703, n);
        if (!ok) return;
        tc_fence_after();
#pragma unroll
        for (int i = 0; i < kUC / 16; ++i) umma_bf16_ts(tO2, tP + i * 8, ahead(v, i * 2048), id_pv, i > 0 ? 1u : 0u);
        umma_commit(o2_full);
        umma_commit(&empty[n & 1]);
      };
      for (int w = blockIdx.x, have; ok && (have = item_at(w, it)) != 0; w += gridDim.x) {
        if (have == 1) continue;
        if (lane == 0) {
          for (int n = k; n < k + it.chunks && ok; ++n) {
            const uint32_t stage = (n & 1) * USmem::kStage;
            const uint64_t q = ahead(d_q, stage), key = ahead(d_k, stage);
            ok = mbar_wait(&full[n & 1], (n >> 1) & 1, abort_flag, p.status, 1701, n);
            if (ok && n > 0) ok = mbar_wait(p_full, (n - 1) & 1, abort_flag, p.status, 1702, n);  // A is free
            if (!ok) break;
            tc_fence_after();
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              if (i >= steps) break;
              const uint32_t off = (i >> 2) * kUTile + (i & 3) * 32;
              umma_bf16_ss(tA, ahead(q, off), ahead(key, off), id_qk, i > 0 ? 1u : 0u);
            }
            umma_commit(a_full);
            if (n > 0) product_pv(n - 1);
          }
        }
        ok = __all_sync(0xffffffffu, ok) != 0;
        k += it.chunks;
      }
      if (lane == 0 && ok && k > 0) {
        ok = mbar_wait(p_full, (k - 1) & 1, abort_flag, p.status, 1702, k);
        if (ok) {
          tc_fence_after();
          product_pv(k - 1);
        }
      }
      __syncwarp();
    }
  } else if (warp == 2) {
    // ------------------------------------------------------------------ O1 = Q S, S += K^T V
    constexpr uint32_t id_kv = make_idesc_bf16(128, 128, true, true), id_qs = make_idesc_bf16(128, 128, false, true);
    const int steps = (p.dk + 15) / 16;
    const uint32_t base = smem_u32(smem);
    const uint64_t d_kt = make_smem_desc(base + USmem::kK, kUTile, 1024), d_values = make_smem_desc(base + USmem::kValues, kUTile, 1024);
    const uint64_t d_q = make_smem_desc(base + USmem::kQ, 16, 1024), d_state = make_smem_desc(base + USmem::kState, kUTile, 1024);
    for (int w = blockIdx.x, have; ok && (have = item_at(w, it)) != 0; w += gridDim.x) {
      if (have == 1) continue;
      if (lane == 0) {
        for (int n = k; n < k + it.chunks; ++n) {
          const uint32_t stage = (n & 1) * USmem::kStage;
          const uint64_t kt = ahead(d_kt, stage), q = ahead(d_q, stage);
          ok = mbar_wait(&full[n & 1], (n >> 1) & 1, abort_flag, p.status, 1704, n) && mbar_wait(s_ready, n & 1, abort_flag, p.status, 1705, n);
          if (!kStateOnly && ok) ok = mbar_wait(o_read, (n & 1) ^ 1, abort_flag, p.status, 1706, n);
          if (!ok) break;
          tc_fence_after();
          if (!kStateOnly) {
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              if (i >= steps) break;
              umma_bf16_ss(tO1, ahead(q, (i >> 2) * kUTile + (i & 3) * 32), ahead(d_state, i * 2048), id_qs, i > 0 ? 1u : 0u);
            }
            umma_commit(o1_full);
          }
          ok = mbar_wait(v_ready, n & 1, abort_flag, p.status, 1707, n);
          if (!ok) break;
          tc_fence_after();
#pragma unroll
          for (int i = 0; i < kUC / 16; ++i) umma_bf16_ss(tS, ahead(kt, i * 2048), ahead(d_values, i * 2048), id_kv, 1u);
          umma_commit(s_full);
          umma_commit(&empty[n & 1]);
        }
      }
      ok = __all_sync(0xffffffffu, ok) != 0;
      k += it.chunks;
    }
  } else if (warp >= 4 && warp < 8) {
    // ------------------------------------------------------------------ weights, then the outputs of the chunk before
    if constexpr (!kStateOnly) {
      float* s_pow = reinterpret_cast<float*>(smem + USmem::kPow);
      {
        uint32_t zero[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) zero[i] = 0u;
        for (int b = quad + 1; b < 4; ++b) tmem_st_32x16(tP + lane_addr + b * 16, zero);
      }
      // outputs of chunk number n: this thread's row (null: past the end), how many columns there are, decay^(row + 1)
      __nv_bfloat16* to = nullptr;
      int cols = 0;
      float to_row = 0.f;
      auto write_outputs = [&](int n) {
        if (!wait_all(o1_full, n & 1, 1711, n) || !wait_all(o2_full, n & 1, 1712, n)) return false;
        tc_fence_after();
#pragma unroll 1
        for (int half = 0; half < 64; half += 32) {
          uint32_t o1[32], lo[32], o2[32];
          tmem_ld_32x32(tO1 + lane_addr + half, o1);
          tmem_ld_32x32(tO1 + 64 + lane_addr + half, lo);
          tmem_ld_32x32(tO2 + lane_addr + half, o2);
          tmem_ld_wait();
          if (half > 0) {
            tc_fence_before();
            arrive(o_read);
          }
#pragma unroll
          for (int i = 0; i < 32; i += 2)
            o1[i / 2] = pack_bf16x2(fmaf(__uint_as_float(o1[i]) + __uint_as_float(lo[i]), to_row, __uint_as_float(o2[i])),
                                    fmaf(__uint_as_float(o1[i + 1]) + __uint_as_float(lo[i + 1]), to_row, __uint_as_float(o2[i + 1])));
          if (to != nullptr) {
#pragma unroll
            for (int u = 0; u < 4; ++u)
              if (half + u * 8 < cols) *reinterpret_cast<uint4*>(to + half + u * 8) = make_uint4(o1[4 * u], o1[4 * u + 1], o1[4 * u + 2], o1[4 * u + 3]);
          }
        }
        return true;
      };
      for (int w = blockIdx.x, have; ok && (have = item_at(w, it)) != 0; w += gridDim.x) {
        if (have == 1) continue;
        const float decay = p.decay[it.h], power = powf(decay, static_cast<float>(row)), item_to_row = power * decay;
        named_bar_sync(1, 128);  // the last item's powers have been read
        s_pow[32 + row] = power * p.key_scale;
        if (warp == 4) s_pow[lane] = 0.f;
        named_bar_sync(1, 128);
        __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (it.r0 + static_cast<long long>(row)) * ldo + it.h * p.dv + it.c0;
        for (int c = 0; c < it.chunks && ok; ++c, ++k) {
          ok = wait_all(a_full, k & 1, 1710, k);
          if (ok && k > 0) ok = wait_all(o2_full, (k - 1) & 1, 1713, k);  // the last P has been read
          if (!ok) break;
          tc_fence_after();
          const float* t = s_pow + 32 + row;  // t[-j]: the weight of key j, zero for later keys
#pragma unroll 1
          for (int b = 0; b <= quad; ++b, t -= 32) {
            uint32_t a[32], x[16];
            tmem_ld_32x32(tA + lane_addr + b * 32, a);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) x[i] = pack_bf16x2(__uint_as_float(a[2 * i]) * t[-2 * i], __uint_as_float(a[2 * i + 1]) * t[-2 * i - 1]);
            tmem_st_32x16(tP + lane_addr + b * 16, x);
          }
          tmem_st_wait();
          tc_fence_before();
          arrive(p_full);
          if (k > 0) ok = write_outputs(k - 1);
          to = row < it.rows - c * kUC ? out + static_cast<long long>(c) * kUC * ldo : nullptr;
          cols = p.dv - it.c0;
          to_row = item_to_row;
        }
      }
      if (ok && k > 0) write_outputs(k - 1);
    }
  } else if (warp >= 8 && warp < 12) {
    // ------------------------------------------------------------------ the state
    const bool used = quad * 32 < p.dk;  // this warp's rows hold keys
    uint8_t* s_state = smem + USmem::kState + row * 128;
    // 32 columns of this thread's row: the sum of the accumulator's halves
    auto read_state = [&](int col, float (&x)[32]) {
      uint32_t t[32], lo[32];
      tmem_ld_32x32(tS + lane_addr + col, t);
      tmem_ld_32x32(tS + 64 + lane_addr + col, lo);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; ++i) x[i] = __uint_as_float(t[i]) + __uint_as_float(lo[i]);
    };
    for (int w = blockIdx.x, have; ok && (have = item_at(w, it)) != 0; w += gridDim.x) {
      if (have == 1) continue;
      const float decay = p.decay[it.h];
      const float whole = powf(decay, static_cast<float>(kUC)), part = powf(decay, static_cast<float>(it.rows - (it.chunks - 1) * kUC));
      float* slot = p.state + (static_cast<long long>(it.s.slot) * p.H + it.h) * head + static_cast<long long>(row) * p.dv + it.c0;
      float* scratch = p.pieces + (static_cast<long long>(it.index) * p.H + it.h) * head + static_cast<long long>(row) * p.dv + it.c0;
      const float* from = kStateOnly || row >= p.dk ? nullptr : it.of > 1 ? scratch : it.s.from_state ? slot : nullptr;
      for (int c = 0; c < it.chunks && ok; ++c, ++k) {
        if (c > 0) ok = wait_all(s_full, (k - 1) & 1, 1720, k);
        if (!kStateOnly && ok && k > 0) ok = wait_all(o1_full, (k - 1) & 1, 1721, k);  // the last chunk's state has been read
        if (!ok) break;
        tc_fence_after();
        const float f = c == it.chunks - 1 ? part : whole;
        if (used) {
#pragma unroll 1
          for (int col = 0; col < 64; col += 32) {
            float x[32];
            if (c > 0) {
              read_state(col, x);
            } else {
#pragma unroll
              for (int i = 0; i < 32; i += 4) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (from != nullptr && it.c0 + col + i < p.dv) v = *reinterpret_cast<const float4*>(from + col + i);
                x[i] = v.x; x[i + 1] = v.y; x[i + 2] = v.z; x[i + 3] = v.w;
              }
            }
            if constexpr (!kStateOnly) {
#pragma unroll
              for (int u = 0; u < 4; ++u) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) split2(x[u * 8 + 2 * e], x[u * 8 + 2 * e + 1], hi[e], lo[e]);
                uint8_t* at = s_state + ((((col >> 3) + u) ^ (row & 7)) << 4);
                *reinterpret_cast<uint4*>(at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                *reinterpret_cast<uint4*>(at + kUTile) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
              }
            }
            uint32_t t[32];
#pragma unroll
            for (int i = 0; i < 32; ++i) t[i] = __float_as_uint(x[i] * f);
            tmem_st_32x32(tS + lane_addr + col, t);
#pragma unroll
            for (int i = 0; i < 32; ++i) t[i] = 0u;
            tmem_st_32x32(tS + 64 + lane_addr + col, t);
          }
          tmem_st_wait();
        }
        fence_proxy_async_smem();
        tc_fence_before();
        arrive(s_ready);
      }
      if (ok) ok = wait_all(s_full, (k - 1) & 1, 1722, k);
      if (ok && used && (kStateOnly || it.piece == it.of - 1)) {
        tc_fence_after();
        float* to = kStateOnly ? scratch : slot;
#pragma unroll 1
        for (int col = 0; col < 64; col += 32) {
          float x[32];
          read_state(col, x);
          if (row < p.dk) {
#pragma unroll
            for (int i = 0; i < 32; i += 4)
              if (it.c0 + col + i < p.dv) *reinterpret_cast<float4*>(to + col + i) = make_float4(x[i], x[i + 1], x[i + 2], x[i + 3]);
          }
        }
      }
    }
  } else if (warp >= 12) {
    // ------------------------------------------------------------------ the decayed values
    uint8_t* s_values = smem + USmem::kValues + row * 128;
    for (int w = blockIdx.x, have; ok && (have = item_at(w, it)) != 0; w += gridDim.x) {
      if (have == 1) continue;
      const float decay = p.decay[it.h];
      const int last = it.rows - (it.chunks - 1) * kUC;
      const float whole = powf(decay, static_cast<float>(kUC - 1 - row)) * p.key_scale;
      const float part = row < last ? powf(decay, static_cast<float>(last - 1 - row)) * p.key_scale : 0.f;
      for (int c = 0; c < it.chunks; ++c, ++k) {
        const int n = c == it.chunks - 1 ? last : kUC;
        const float f = c == it.chunks - 1 ? part : whole;
        ok = wait_all(&full[k & 1], (k >> 1) & 1, 1731, k);
        if (ok && k > 0) ok = wait_all(s_full, (k - 1) & 1, 1730, k);  // the last chunk's values have been read
        if (!ok) break;
        const uint8_t* v = smem + (k & 1) * USmem::kStage + USmem::kV + row * 128;
#pragma unroll 1
        for (int u = 0; u < 8; u += 2) {
          const int at = (u ^ (row & 7)) << 4;  // the next unit lies at at ^ 16
          uint4 y[2];
          y[0] = *reinterpret_cast<const uint4*>(v + at);
          y[1] = *reinterpret_cast<const uint4*>(v + (at ^ 16));
          if (row >= n) y[0] = y[1] = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const uint32_t in[4] = {y[j].x, y[j].y, y[j].z, y[j].w};
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&in[e]));
              split2(z.x * f, z.y * f, hi[e], lo[e]);
            }
            uint8_t* dst = s_values + (at ^ (j << 4));
            *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(dst + kUTile) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
        }
        fence_proxy_async_smem();
        arrive(v_ready);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc<512>(tmem);
  }
}

int run_umma(const Params& p, int items, cudaStream_t s) {
  CUtensorMap tmQ, tmK, tmV;
  int rc = make_tmap_heads_bf16(&tmQ, p.q, p.T, p.H, p.dk, p.ld, kUC);
  if (rc == kErrOk) rc = make_tmap_heads_bf16(&tmK, p.k, p.T, p.H, p.dk, p.ld, kUC);
  if (rc == kErrOk) rc = make_tmap_heads_bf16(&tmV, p.v, p.T, p.H, p.dv, p.ld, kUC);
  if (rc != kErrOk) return rc;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(umma_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, USmem::kTotal) != cudaSuccess ||
        cudaFuncSetAttribute(umma_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, USmem::kTotal) != cudaSuccess)
      return kErrCuda;
    attr_set = true;
  }
  const long long all = static_cast<long long>(items) * p.H * ((p.dv + 63) / 64);
  if (all > 0x3fffffff) return kErrTooLarge;
  const int grid = static_cast<int>(all < num_sms() ? all : num_sms());
  if (p.pieces != nullptr) {
    umma_kernel<true><<<grid, kUThreads, USmem::kTotal, s>>>(tmQ, tmK, tmV, p);
    carry_states(p, s);
  }
  umma_kernel<false><<<grid, kUThreads, USmem::kTotal, s>>>(tmQ, tmK, tmV, p);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

}  // namespace linattn
}  // namespace lvb
