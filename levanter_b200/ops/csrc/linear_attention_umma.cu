// The chunked form of linear attention with fixed decays (linear_attention.cu says what it computes) for keys of up to 128, on tcgen05.
//
// A CTA walks one piece of one head in chunks of 128 rows, for 64 columns of the values.  Per chunk, with the state S [dk, 64] as an fp32
// accumulator in tensor memory:
//   A = Q K^T (128 x 128)        -> P = A o decays, bf16, in tensor memory again (row i, keys up to i; the rest stays zero)
//   O1 = Q [S_hi | S_lo]         S is written to shared memory in two bf16 parts, side by side, before the chunk touches it
//   O2 = P V,  out = decay^(i+1) (O1_hi + O1_lo) + O2
//   S <- decay^n S + K^T [V_hi | V_lo]   with the decayed values in two bf16 parts, and S the sum of the two halves of its accumulator
// Side by side the two parts are one MMA of 128 columns, which reads the other factor once.  Warp 0 fetches Q, K and V by TMA two chunks
// deep, warp 1 issues the MMAs, warps 2-5 make P and write the outputs, warps 6-9 carry the state and decay the values.
// TMEM map (512 columns): A [0, 128)  P [128, 192)  O2 [192, 256)  O1 [256, 384)  S [384, 512).
#include "linear_attention.cuh"

namespace lvb {
namespace linattn {

constexpr int kUC = 128;             // rows of a chunk
constexpr int kUThreads = 320;
constexpr int kUTile = 128 * 64 * 2; // 128 rows of 64 columns

struct USmem {
  static constexpr int kQ = 0, kK = 2 * kUTile, kV = 4 * kUTile;  // within a stage
  static constexpr int kStage = 5 * kUTile;
  static constexpr int kState = 2 * kStage;      // S in two parts
  static constexpr int kValues = kState + 2 * kUTile;  // decayed V in two parts
  static constexpr int kPow = kValues + 2 * kUTile;    // decay^0 .. decay^128
  static constexpr int kBars = kPow + (kUC + 4) * 4;
  static constexpr int kNumBars = 11;
  static constexpr int kTotal = kBars + kNumBars * 8 + 16 + 1024;
};
static_assert(USmem::kTotal <= 227 * 1024 && USmem::kBars % 8 == 0, "shared memory of one CTA");

// kStateOnly: what a piece adds to a zero state, for all pieces but the last of a sequence.
template <bool kStateOnly>
__global__ void __launch_bounds__(kUThreads, 1)
umma_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int h = blockIdx.y, c0 = blockIdx.z * 64;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long ldo = static_cast<long long>(p.H) * p.dv;
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + h * p.dv + c0;
  int seq = 0, piece = 0, of = 0;
  if (!find_piece(p, blockIdx.x, seq, piece, of)) {
    if constexpr (!kStateOnly) {  // the work items past the last piece (there is always one): zeros for the rows of no sequence
      const int n_seq = live_sequences(p);
      const int cols = min(p.dv - c0, 64);
      for (int r = (n_seq > 0 ? p.cu_q_lens[n_seq] : 0) + blockIdx.x - of; r < p.T; r += gridDim.x - of)
        for (int e = threadIdx.x; e < cols; e += kUThreads) out[r * ldo + e] = __float2bfloat16(0.f);
    }
    return;
  }
  Sequence s;
  if (!sequence(p, seq, s)) return;
  if (kStateOnly && piece == of - 1) return;
  const int r0 = s.r0 + piece * p.piece, rows = min(p.piece, s.r1 - r0), chunks = (rows + kUC - 1) / kUC;
  const int ck = (p.dk + 63) / 64;  // 64-column parts of queries and keys

  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + USmem::kBars);
  uint64_t* full = bars;          // [2 stages]
  uint64_t* empty = bars + 2;     // [2 stages]
  uint64_t* a_full = bars + 4;    // A is complete, and so is everything issued before
  uint64_t* p_full = bars + 5;    // P is in place
  uint64_t* s_ready = bars + 6;   // the state has been read out, written to shared memory and decayed
  uint64_t* v_ready = bars + 7;   // the decayed values are in place
  uint64_t* s_full = bars + 8;    // the state has taken up the chunk
  uint64_t* o_full = bars + 9;    // the chunk's outputs are complete
  uint64_t* o_read = bars + 10;   // and have been read out
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bars + USmem::kNumBars);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);
  float* s_pow = reinterpret_cast<float*>(smem + USmem::kPow);
  const float decay = p.decay[h];
  for (int t = threadIdx.x; t <= kUC; t += kUThreads) s_pow[t] = powf(decay, static_cast<float>(t));
  if (threadIdx.x == 0) {
    *abort_flag = 0;
    for (int i = 0; i < USmem::kNumBars; ++i) mbar_init(&bars[i], i == 5 || i == 6 || i == 7 || i == 10 ? 4 : 1);  // four warps, or one thread
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
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;
  const uint32_t tA = tmem, tP = tmem + 128, tO2 = tmem + 192, tO1 = tmem + 256, tS = tmem + 384;
  const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
  const int row = (warp & 3) * 32 + lane;
  auto rows_of = [&](int c) { return min(rows - c * kUC, kUC); };
  // for warps that go on to collective instructions: all lanes or none
  auto wait_all = [&](uint64_t* bar, uint32_t parity, int site, int extra) {
    return __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag, p.status, site, extra)) != 0;
  };

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      bool ok = true;
      int issued = 0;
      for (int c = 0; c < chunks && ok; ++c) {
        const int st = c & 1;
        ok = mbar_wait(&empty[st], ((c >> 1) & 1) ^ 1, abort_flag, p.status, 1700, c);
        if (!ok) break;
        uint8_t* at = smem + st * USmem::kStage;
        mbar_expect_tx(&full[st], ((kStateOnly ? 1 : 2) * ck + 1) * kUTile);
        for (int i = 0; i < ck; ++i) {
          if (!kStateOnly) tma_load_3d(at + USmem::kQ + i * kUTile, &tmQ, &full[st], 64 * i, h, r0 + c * kUC);
          tma_load_3d(at + USmem::kK + i * kUTile, &tmK, &full[st], 64 * i, h, r0 + c * kUC);
        }
        tma_load_3d(at + USmem::kV, &tmV, &full[st], c0, h, r0 + c * kUC);
        ++issued;
      }
      if (!ok)  // let the copies in flight land
        for (int c = max(issued - 2, 0); c < issued; ++c) mbar_wait_quiet(&full[c & 1], (c >> 1) & 1);
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      constexpr uint32_t id_qk = make_idesc_bf16(128, 128, false, false);
      // the second factor by rows of the inner index: Q S, P V, and (the first one too) K^T V
      constexpr uint32_t id_qs = make_idesc_bf16(128, 128, false, true);
      constexpr uint32_t id_pv = make_idesc_bf16(128, 64, false, true);
      constexpr uint32_t id_kv = make_idesc_bf16(128, 128, true, true);
      const int steps = (p.dk + 15) / 16;
      const uint32_t base = smem_u32(smem);
      auto product_qk = [&](int st) {
        const uint32_t q = base + st * USmem::kStage + USmem::kQ, k = base + st * USmem::kStage + USmem::kK;
        for (int i = 0; i < steps; ++i) {
          const uint32_t off = (i >> 2) * kUTile + (i & 3) * 32;
          umma_bf16_ss(tA, make_smem_desc(q + off, 16, 1024), make_smem_desc(k + off, 16, 1024), id_qk, i > 0 ? 1u : 0u);
        }
        umma_commit(a_full);
      };
      bool ok = mbar_wait(&full[0], 0, abort_flag, p.status, 1701, 0);
      if (ok) {
        tc_fence_after();
        if (!kStateOnly) product_qk(0);
      }
      for (int c = 0; c < chunks && ok; ++c) {
        const int st = c & 1;
        const uint32_t stage = base + st * USmem::kStage;
        ok = mbar_wait(s_ready, c & 1, abort_flag, p.status, 1702, c);
        if (!ok) break;
        if (!kStateOnly) {
          ok = mbar_wait(o_read, (c & 1) ^ 1, abort_flag, p.status, 1703, c);
          if (!ok) break;
          tc_fence_after();
          for (int i = 0; i < steps; ++i)
            umma_bf16_ss(tO1, make_smem_desc(stage + USmem::kQ + (i >> 2) * kUTile + (i & 3) * 32, 16, 1024),
                         make_smem_desc(base + USmem::kState + i * 2048, kUTile, 1024), id_qs, i > 0 ? 1u : 0u);
        }
        ok = mbar_wait(v_ready, c & 1, abort_flag, p.status, 1704, c);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int i = 0; i < kUC / 16; ++i)
          umma_bf16_ss(tS, make_smem_desc(stage + USmem::kK + i * 2048, kUTile, 1024), make_smem_desc(base + USmem::kValues + i * 2048, kUTile, 1024),
                       id_kv, 1u);
        umma_commit(s_full);
        if (!kStateOnly) {
          ok = mbar_wait(p_full, c & 1, abort_flag, p.status, 1705, c);
          if (!ok) break;
          tc_fence_after();
#pragma unroll
          for (int i = 0; i < kUC / 16; ++i)
            umma_bf16_ts(tO2, tP + i * 8, make_smem_desc(stage + USmem::kV + i * 2048, kUTile, 1024), id_pv, i > 0 ? 1u : 0u);
          umma_commit(o_full);
        }
        umma_commit(&empty[st]);
        if (c + 1 < chunks) {
          ok = mbar_wait(&full[st ^ 1], ((c + 1) >> 1) & 1, abort_flag, p.status, 1706, c);
          if (!ok) break;
          tc_fence_after();
          if (!kStateOnly) product_qk(st ^ 1);
        }
      }
    }
  } else if (warp < 6) {
    // ------------------------------------------------------------------ weights and outputs
    if constexpr (!kStateOnly) {
      const int quad = warp & 3;
      {
        uint32_t zero[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) zero[i] = 0u;
        for (int b = quad + 1; b < 4; ++b) tmem_st_32x16(tP + lane_addr + b * 16, zero);
      }
      const float to_row = s_pow[row + 1];
      // decay^(i - j) for the 32 keys of a block: on the diagonal directly (zero for later keys), before it as decay^(i - last key) times
      // decay^(last key - j)
      float diagonal[32], to_last[32];
#pragma unroll
      for (int j = 0; j < 32; ++j) {
        const float f = s_pow[max(lane - j, 0)] * p.key_scale;
        diagonal[j] = j <= lane ? f : 0.f;
        to_last[j] = s_pow[31 - j];
      }
      bool ok = true;
      for (int c = 0; c < chunks && ok; ++c) {
        const int n = rows_of(c);
        ok = wait_all(a_full, c & 1, 1710, c);
        if (!ok) break;
        tc_fence_after();
#pragma unroll 1
        for (int b = 0; b <= quad; ++b) {
          uint32_t a[32], w[16];
          tmem_ld_32x32(tA + lane_addr + b * 32, a);
          tmem_ld_wait();
          if (b < quad) {
            const float f = s_pow[row - b * 32 - 31] * p.key_scale;
#pragma unroll
            for (int i = 0; i < 16; ++i)
              w[i] = pack_bf16x2(__uint_as_float(a[2 * i]) * to_last[2 * i] * f, __uint_as_float(a[2 * i + 1]) * to_last[2 * i + 1] * f);
          } else {
#pragma unroll
            for (int i = 0; i < 16; ++i) w[i] = pack_bf16x2(__uint_as_float(a[2 * i]) * diagonal[2 * i], __uint_as_float(a[2 * i + 1]) * diagonal[2 * i + 1]);
          }
          tmem_st_32x16(tP + lane_addr + b * 16, w);
        }
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(p_full);
        ok = wait_all(o_full, c & 1, 1711, c);
        if (!ok) break;
        tc_fence_after();
        __nv_bfloat16* to = out + static_cast<long long>(r0 + c * kUC + row) * ldo;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t o1[32], lo[32], o2[32];
          tmem_ld_32x32(tO1 + lane_addr + half * 32, o1);
          tmem_ld_32x32(tO1 + 64 + lane_addr + half * 32, lo);
          tmem_ld_32x32(tO2 + lane_addr + half * 32, o2);
          tmem_ld_wait();
          if (half == 1) {
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(o_read);
          }
          if (row < n) {
#pragma unroll
            for (int u = 0; u < 4; ++u) {
              if (c0 + half * 32 + u * 8 >= p.dv) continue;
              uint32_t w[4];
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const int i = u * 8 + 2 * e;
                w[e] = pack_bf16x2(fmaf(__uint_as_float(o1[i]) + __uint_as_float(lo[i]), to_row, __uint_as_float(o2[i])),
                                   fmaf(__uint_as_float(o1[i + 1]) + __uint_as_float(lo[i + 1]), to_row, __uint_as_float(o2[i + 1])));
              }
              *reinterpret_cast<uint4*>(to + half * 32 + u * 8) = make_uint4(w[0], w[1], w[2], w[3]);
            }
          }
        }
      }
    }
  } else {
    // ------------------------------------------------------------------ the state and the decayed values
    const long long head = static_cast<long long>(p.dk) * p.dv;
    float* slot = p.state + (static_cast<long long>(s.slot) * p.H + h) * head + static_cast<long long>(row) * p.dv + c0;
    float* scratch = p.pieces + (static_cast<long long>(blockIdx.x) * p.H + h) * head + static_cast<long long>(row) * p.dv + c0;
    const bool used = (warp & 3) * 32 < p.dk;  // this warp's rows hold keys
    float x[64];
#pragma unroll
    for (int i = 0; i < 64; ++i) x[i] = 0.f;
    if constexpr (!kStateOnly) {
      const float* from = of > 1 ? scratch : s.from_state ? slot : nullptr;
      if (from != nullptr && row < p.dk) {
#pragma unroll
        for (int i = 0; i < 64; i += 4) {
          if (c0 + i >= p.dv) continue;
          const float4 v = *reinterpret_cast<const float4*>(from + i);
          x[i] = v.x; x[i + 1] = v.y; x[i + 2] = v.z; x[i + 3] = v.w;
        }
      }
    }
    auto read_state = [&] {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t t[32], lo[32];
        tmem_ld_32x32(tS + lane_addr + half * 32, t);
        tmem_ld_32x32(tS + 64 + lane_addr + half * 32, lo);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) x[half * 32 + i] = __uint_as_float(t[i]) + __uint_as_float(lo[i]);
      }
    };
    uint8_t* s_state = smem + USmem::kState + row * 128;
    uint8_t* s_values = smem + USmem::kValues + row * 128;
    bool ok = true;
    for (int c = 0; c < chunks && ok; ++c) {
      const int st = c & 1, n = rows_of(c);
      if (c > 0) {
        ok = wait_all(s_full, (c - 1) & 1, 1720, c);
        if (!ok) break;
        tc_fence_after();
        if (used) read_state();
      }
      if (used) {
        if constexpr (!kStateOnly) {
#pragma unroll
          for (int u = 0; u < 8; ++u) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) split2(x[u * 8 + 2 * e], x[u * 8 + 2 * e + 1], hi[e], lo[e]);
            uint8_t* at = s_state + ((u ^ (row & 7)) << 4);
            *reinterpret_cast<uint4*>(at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(at + kUTile) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
        }
        const float f = s_pow[n];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t t[32];
#pragma unroll
          for (int i = 0; i < 32; ++i) t[i] = __float_as_uint(x[half * 32 + i] * f);
          tmem_st_32x32(tS + lane_addr + half * 32, t);
#pragma unroll
          for (int i = 0; i < 32; ++i) t[i] = 0u;
          tmem_st_32x32(tS + 64 + lane_addr + half * 32, t);
        }
        tmem_st_wait();
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(s_ready);
      ok = wait_all(&full[st], (c >> 1) & 1, 1721, c);
      if (!ok) break;
      const uint8_t* v = smem + st * USmem::kStage + USmem::kV + row * 128;
      const float f = row < n ? s_pow[max(n - 1 - row, 0)] * p.key_scale : 0.f;
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const int at = (u ^ (row & 7)) << 4;
        uint4 w = *reinterpret_cast<const uint4*>(v + at);
        if (row >= n) w = make_uint4(0u, 0u, 0u, 0u);
        const uint32_t in[4] = {w.x, w.y, w.z, w.w};
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&in[e]));
          split2(y.x * f, y.y * f, hi[e], lo[e]);
        }
        *reinterpret_cast<uint4*>(s_values + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(s_values + at + kUTile) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(v_ready);
    }
    if (ok) ok = wait_all(s_full, (chunks - 1) & 1, 1722, chunks);
    if (ok && used && (kStateOnly || piece == of - 1)) {
      tc_fence_after();
      read_state();
      float* to = kStateOnly ? scratch : slot;
      if (row < p.dk) {
#pragma unroll
        for (int i = 0; i < 64; i += 4)
          if (c0 + i < p.dv) *reinterpret_cast<float4*>(to + i) = make_float4(x[i], x[i + 1], x[i + 2], x[i + 3]);
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
  const dim3 grid(items, p.H, (p.dv + 63) / 64);
  if (p.pieces != nullptr) {
    umma_kernel<true><<<grid, kUThreads, USmem::kTotal, s>>>(tmQ, tmK, tmV, p);
    carry_states(p, s);
  }
  umma_kernel<false><<<grid, kUThreads, USmem::kTotal, s>>>(tmQ, tmK, tmV, p);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

}  // namespace linattn
}  // namespace lvb
