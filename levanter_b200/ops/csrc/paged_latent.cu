// Latent attention over a paged cache, in the form in which every query head reads the same row per key: the row [c, k] of a key holds a
// compressed part c (rank elements) and a key part k shared by the heads, the query of head h is [W_uk(h)^T q, q'], the score is
// the product of the two rows, and the value is c itself (the caller applies W_uv(h) to the result).  So a key is read once for
// all heads and used twice.
//
//  * paged_latent: one CTA per (packed query row, group of up to 32 query heads, partition of the visible keys).  The keys come
//    by TMA in tiles of 64 rows (128-byte swizzle; boxes of the rows of a page, at most 64), two to four tiles deep.  Eight warps
//    compute: scores are warp-level MMAs (m16n8k16, bf16, fp32 accumulation) with the
//    query heads as the M rows, a warp taking 32 keys and a quarter of the row; then every warp owns the online softmax of a few
//    heads, which adds up the quarters; then a set of 16-column pieces of the output, with the value operand read from the key
//    tile by transposing ldmatrix.  Shared-memory reads bound a tile as much as its transfer does, hence the large share per
//    warp.  The visible keys of a row are cut evenly over the partitions inside the kernel, so the launch needs no lengths from
//    the device; a second kernel merges the partitions.
//  * head_product: out(t, h) = A(t, h) B(h) or A(t, h) B(h)^T for every head: the two products with per-head weights around it.
#include "common.cuh"

namespace lvb {
namespace latent {

constexpr int kWarps = 8;              // computing warps
constexpr int kThreads = kWarps * 32;
// A ninth warp is the producer, except where two M tiles and a long row want all registers that eight warps can have: there the first
// computing warp issues the copies.
__host__ __device__ constexpr bool has_producer(int m_tiles, int pieces) { return m_tiles == 1 || pieces <= 2; }
__host__ __device__ constexpr int cta_threads(int m_tiles, int pieces) { return kThreads + (has_producer(m_tiles, pieces) ? 32 : 0); }
constexpr int kSplit = 4;      // parts that the inner dimension of the scores is cut into
constexpr int kMaxStages = 4;
constexpr int kMaxSmem = 226 * 1024;
constexpr int kTileKeys = 64;
constexpr int kMinPart = 64;   // keys of a partition, at least
constexpr int kMaxRank = 512;
constexpr int kScoreLd = 68;   // floats per row of the score tile
constexpr int kProbLd = 72;    // bf16 per row of the probability tile

__device__ __forceinline__ void cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void ldm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldm_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct Params {
  const __nv_bfloat16* q;         // [T, H, width]
  const __nv_bfloat16* kv_pages;  // [num_pages, page_size, width]
  const int *kv_lens, *page_indices, *cu_q_lens, *num_seqs;
  const float* sink;              // optional [H]: joins the softmax denominator of its head as it is
  __nv_bfloat16* out;             // [T, H, rank]
  float* part_o;                  // [T, H, parts, rank]
  float* part_ml;                 // [T, H, parts, 2]: maximum (base 2) and sum
  int T, H, width, rank, S, pages_per_seq, page_size, num_pages, parts, window, stages;
  float scale;
  int* status;
  int box;   // rows of a TMA box: a power of two that divides the page size and 64
  int box_log;
  int whole; // a box holds whole rows [box][chunks][128 bytes]; else all their chunks [chunks][box][128 bytes] (grouped) or one [box][128 bytes]
  int grouped;
};

__device__ __forceinline__ bool locate(const Params& p, int t, int& seq, int& ctx) {
  int n = p.num_seqs[0];
  n = n < p.S ? n : p.S;
  if (n <= 0 || t >= p.cu_q_lens[n]) return false;
  int lo = 0, hi = n;
  while (lo < hi) {
    const int mid = (lo + hi) >> 1;
    if (p.cu_q_lens[mid + 1] > t) hi = mid; else lo = mid + 1;
  }
  seq = lo;
  const int kl = p.kv_lens[seq];
  if (kl <= 0 || kl > p.pages_per_seq * p.page_size) return false;
  ctx = kl - p.cu_q_lens[seq + 1] + t + 1;  // the row's position + 1
  return ctx > 0;
}

// Visible keys [first, ctx) of a row, and the keys of one partition (a multiple of the tile).
__device__ __forceinline__ int first_key(const Params& p, int ctx) { return p.window > 0 && ctx > p.window ? ctx - p.window : 0; }
__device__ __forceinline__ int part_keys(const Params& p, int visible) {
  const int even = (visible + p.parts - 1) / p.parts;
  const int n = even > kMinPart ? even : kMinPart;
  return (n + kTileKeys - 1) / kTileKeys * kTileKeys;
}

// What head h's sink adds to a softmax sum relative to the maximum m (base 2).  Far above the maximum it is infinite and the output zero.
__device__ __forceinline__ float sink_term(const Params& p, int h, float m) { return exp2f(p.sink[h] * 1.4426950408889634f - m); }

// Key tiles are cut into chunks of 64 columns (128 bytes); columns past the width are zeros.
__host__ __device__ constexpr int chunks_of(int width) { return (width + 63) / 64; }
__host__ __device__ constexpr int stage_bytes(int width) { return chunks_of(width) * kTileKeys * 128; }
__host__ __device__ constexpr int row_bytes(int width) { return chunks_of(width) * 128 + 16; }  // of a staged query: an odd multiple of 16
// key tiles (1024-byte aligned), queries, partial score tiles, probabilities, three numbers per head, barriers
__host__ __device__ constexpr int smem_bytes(int m_tiles, int width, int stages) {
  return 1024 + stages * stage_bytes(width) + m_tiles * 16 * (row_bytes(width) + kSplit * kScoreLd * 4 + kProbLd * 2 + 3 * 4) + 2 * kMaxStages * 8 + 16;
}

// kM: M tiles (16 query heads each) per CTA.  kPieces: 16-column output pieces per warp, at most: rank <= kPieces * 8 * 16.
template <int kM, int kPieces>
__global__ void __launch_bounds__(cta_threads(kM, kPieces), 1) paged_latent_kernel(const __grid_constant__ CUtensorMap tm, Params p) {
  constexpr int kHeads = kM * 16, kCta = cta_threads(kM, kPieces);
  constexpr bool kProducer = has_producer(kM, kPieces);
  constexpr int kRowLanes = 16 / kM;             // lanes per head in the softmax: a warp owns 2 kM heads
  constexpr int kLaneKeys = kTileKeys / kRowLanes;
  extern __shared__ uint8_t smem_raw[];
  const int chunks = chunks_of(p.width), rowb = row_bytes(p.width), stageb = stage_bytes(p.width);
  uint8_t* s_k = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));  // [stages][64 / box][chunks][box][128]
  uint8_t* s_q = s_k + p.stages * stageb;                                      // [kHeads][row]
  float* s_s = reinterpret_cast<float*>(s_q + kHeads * rowb);                  // [kSplit][kHeads][kScoreLd]
  __nv_bfloat16* s_p = reinterpret_cast<__nv_bfloat16*>(s_s + kSplit * kHeads * kScoreLd);  // [kHeads][kProbLd]
  float* s_alpha = reinterpret_cast<float*>(s_p + kHeads * kProbLd);           // [kHeads]
  float* s_m = s_alpha + kHeads;
  float* s_l = s_m + kHeads;
  uint64_t* full = reinterpret_cast<uint64_t*>(s_l + kHeads);  // [kMaxStages]
  uint64_t* empty = full + kMaxStages;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(empty + kMaxStages);
  const int t = blockIdx.x, h0 = blockIdx.y * kHeads, part = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int heads = min(kHeads, p.H - h0);

  int seq = 0, ctx = 0;
  const bool live = locate(p, t, seq, ctx);
  const int first = live ? first_key(p, ctx) : 0;
  const int base = first & ~(p.box - 1);  // whole boxes: the keys before `first` are masked
  const int per = live ? part_keys(p, ctx - base) : 0;
  const int k0 = base + part * per;
  if (!live || k0 >= ctx) {
    if (!live && part == 0) {
      for (int i = threadIdx.x; i < heads * p.rank; i += kCta)
        p.out[(static_cast<long long>(t) * p.H + h0) * p.rank + i] = __float2bfloat16(0.f);
    }
    return;
  }
  const int nk = min(per, ctx - k0);
  const int tiles = (nk + kTileKeys - 1) / kTileKeys;
  const int below = first - k0;  // keys of the partition that come before the window (or <= 0)

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    for (int i = 0; i < p.stages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], kWarps);
    }
    mbar_fence_init();
    tma_prefetch_desc(&tm);
  }
  // queries; rows beyond the heads and columns beyond the width are zeros
  for (int i = threadIdx.x; i < kHeads * chunks * 8; i += kCta) {
    const int r = i / (chunks * 8), c = i - r * (chunks * 8);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < heads && c * 8 < p.width) v = *reinterpret_cast<const uint4*>(p.q + (static_cast<long long>(t) * p.H + h0 + r) * p.width + c * 8);
    *reinterpret_cast<uint4*>(s_q + r * rowb + c * 16) = v;
  }
  __syncthreads();

  // ---- copies: a lane per box
  const int per_group = p.whole || p.grouped ? 1 : chunks, boxes = kTileKeys / p.box * per_group, boxb = p.box * 128 * (chunks / per_group);
  auto lookup = [&](int tile, int i) -> int {  // cache row of box i; past the last key any rows will do, they are masked
    const int key = k0 + tile * kTileKeys + i / per_group * p.box;
    if (i >= boxes || key >= ctx) return 0;
    const int page = p.page_indices[seq * p.pages_per_seq + key / p.page_size];
    return page >= 0 && page < p.num_pages ? page * p.page_size + key % p.page_size : 0;
  };
  auto issue = [&](int tile, int stage, int row_first) {
    if (tile >= tiles) return;
    if (lane == 0) mbar_expect_tx(&full[stage], stageb);
    __syncwarp();
    for (int i = lane; i < boxes; i += 32) {
      const int row = i == lane ? row_first : lookup(tile, i);
      uint8_t* dst = s_k + stage * stageb + i * boxb;
      if (p.whole) tma_load_3d(dst, &tm, &full[stage], 0, 0, row);
      else if (p.grouped) tma_load_3d(dst, &tm, &full[stage], 0, row, 0);
      else tma_load_2d(dst, &tm, &full[stage], i % chunks * 64, row);
    }
  };
  if (kProducer && warp == kWarps) {
    int st = 0;
    uint32_t phase = 0;
    for (int it = 0; it < tiles; ++it) {
      const int row_first = lookup(it, lane);
      bool ok = mbar_wait(&empty[st], phase ^ 1, abort_flag, p.status, 1500, it);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      issue(it, st, row_first);
      if (++st == p.stages) {
        st = 0;
        phase ^= 1;
      }
    }
    return;
  }
  int row_next = 0;
  if (!kProducer && warp == 0) {
    for (int i = 0; i < p.stages - 1; ++i) issue(i, i, lookup(i, lane));
    row_next = lookup(p.stages - 1, lane);
  }

  const float sc_log2 = p.scale * 1.4426950408889634f;
  const int out_pieces = (p.rank + 15) / 16;
  // this warp's part of the scores: 32 keys and a range of k-steps, for all heads
  const int keys_at = (warp & 1) * 32, kpart = warp >> 1;
  const int ks_lo = chunks * 4 * kpart / kSplit, ks_hi = chunks * 4 * (kpart + 1) / kSplit;
  // A 16-byte unit u of row r and chunk c of a tile lies at row_at(r) + c * chunkb, its place in the 128 bytes xor'ed with the
  // number of that 128-byte line (the TMA swizzle).
  const int chunkb = p.whole ? 128 : p.box * 128;
  auto row_at = [&](int r) { return p.whole ? r * chunks * 128 : (r >> p.box_log) * chunks * chunkb + (r & (p.box - 1)) * 128; };
  float* my_scores = s_s + (kpart * kHeads + (lane >> 2)) * kScoreLd + keys_at + (lane & 3) * 2;
  int key_at[2];
#pragma unroll
  for (int j = 0; j < 2; ++j) key_at[j] = row_at(keys_at + j * 16 + (lane >> 4) * 8 + (lane & 7));
  const int val_row = ((lane >> 3) & 1) * 8 + (lane & 7);
  // this lane's part of the softmax: keys lk .. lk + kLaneKeys of head row
  const int row = warp * 2 * kM + lane / kRowLanes, lk = (lane % kRowLanes) * kLaneKeys;
  float m_run = -INFINITY, l_run = 0.f;
  float o[kPieces][kM][2][4];
#pragma unroll
  for (int a = 0; a < kPieces; ++a)
#pragma unroll
    for (int b = 0; b < kM; ++b)
#pragma unroll
      for (int c = 0; c < 4; ++c) { o[a][b][0][c] = 0.f; o[a][b][1][c] = 0.f; }

  int st = 0;
  uint32_t phase = 0;
  for (int it = 0; it < tiles; ++it) {
    if (!kProducer && warp == 0) {  // once everyone is done with the tile before this one, its buffer takes the next copies
      const int prev = st == 0 ? p.stages - 1 : st - 1;
      bool ok = it == 0 || mbar_wait(&empty[prev], st == 0 ? phase ^ 1 : phase, abort_flag, p.status, 1500, it);
      ok = __all_sync(0xffffffffu, ok);
      if (ok) issue(it + p.stages - 1, prev, row_next);
      row_next = lookup(it + p.stages, lane);
    }
    // after a wait that ran out the loop goes on without data, so that everyone still meets at the barriers
    mbar_wait(&full[st], phase, abort_flag, p.status, 1501, it);
    __syncwarp();
    const uint32_t kb = smem_u32(s_k + st * stageb);
    if (it == tiles - 1 && (nk & (kTileKeys - 1)) != 0) {
      // what lies past the last key was never a key of this sequence: 0 * NaN would poison the output
      const int r0 = nk & (kTileKeys - 1);
      for (int i = threadIdx.x; i < (kTileKeys - r0) * chunks * 8; i += kThreads) {
        const int r = r0 + i / (chunks * 8), c = i % (chunks * 8);
        *reinterpret_cast<uint4*>(s_k + st * stageb + row_at(r) + (c >> 3) * chunkb + (c & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
      }
      named_bar_sync(1, kThreads);
    }
    {
      float acc[kM][4][4];
#pragma unroll
      for (int m = 0; m < kM; ++m)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int c = 0; c < 4; ++c) acc[m][j][c] = 0.f;
      const uint32_t qa = smem_u32(s_q) + (lane & 15) * rowb + (lane >> 4) * 16;
      const int unit = (lane >> 3) & 1;
      struct Frags {
        uint32_t a[kM][4], b[2][4];
      } f0, f1;
      auto load = [&](int ks, Frags& f) {
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int line = key_at[j] + (ks >> 2) * chunkb;
          // (keys 0-7, k 0-7), (keys 0-7, k 8-15), (keys 8-15, k 0-7), (keys 8-15, k 8-15)
          ldm_x4(kb + line + ((((ks & 3) * 2 + unit) ^ ((line >> 7) & 7)) << 4), f.b[j][0], f.b[j][1], f.b[j][2], f.b[j][3]);
        }
#pragma unroll
        for (int m = 0; m < kM; ++m) ldm_x4(qa + m * 16 * rowb + ks * 32, f.a[m][0], f.a[m][1], f.a[m][2], f.a[m][3]);
      };
      auto mul = [&](Frags& f) {
#pragma unroll
        for (int m = 0; m < kM; ++m)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            mma16816(acc[m][2 * j], f.a[m], f.b[j][0], f.b[j][1]);
            mma16816(acc[m][2 * j + 1], f.a[m], f.b[j][2], f.b[j][3]);
          }
      };
      load(ks_lo, f0);
      int ks = ks_lo;
#pragma unroll 1
      for (; ks + 1 < ks_hi; ks += 2) {  // the next step's fragments are read ahead
        load(ks + 1, f1);
        mul(f0);
        if (ks + 2 < ks_hi) load(ks + 2, f0);
        mul(f1);
      }
      if (ks < ks_hi) mul(f0);
#pragma unroll
      for (int m = 0; m < kM; ++m)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          *reinterpret_cast<float2*>(my_scores + m * 16 * kScoreLd + j * 8) = make_float2(acc[m][j][0], acc[m][j][1]);
          *reinterpret_cast<float2*>(my_scores + (m * 16 + 8) * kScoreLd + j * 8) = make_float2(acc[m][j][2], acc[m][j][3]);
        }
    }
    named_bar_sync(1, kThreads);
    // the value operand of the warp's first output piece: (keys 0-7, columns 0-7), (keys 8-15, same), (keys 0-7, columns 8-15),
    // (keys 8-15, same) of each 16 keys
    uint32_t vb[4][4];
    auto load_values = [&](int piece) {
#pragma unroll
      for (int h = 0; h < 4; ++h) {
        int r = h * 16 + val_row;
        asm volatile("" : "+r"(r));  // computed per tile: hoisted out of the loop, the addresses would spill
        const int line = row_at(r) + (piece >> 2) * chunkb, unit = (piece & 3) * 2 + (lane >> 4);
        ldm_x4_trans(kb + line + ((unit ^ ((line >> 7) & 7)) << 4), vb[h][0], vb[h][1], vb[h][2], vb[h][3]);
      }
    };
    if (warp < out_pieces) load_values(warp);
    {
      float v[kLaneKeys];
#pragma unroll
      for (int i = 0; i < kLaneKeys; ++i) v[i] = 0.f;
#pragma unroll
      for (int k = 0; k < kSplit; ++k) {
        const float* src = s_s + (k * kHeads + row) * kScoreLd + lk;
#pragma unroll
        for (int i = 0; i < kLaneKeys; i += 4) {
          const float4 x = *reinterpret_cast<const float4*>(src + i);
          v[i] += x.x;
          v[i + 1] += x.y;
          v[i + 2] += x.z;
          v[i + 3] += x.w;
        }
      }
      const int left = nk - it * kTileKeys - lk, hidden = below - it * kTileKeys - lk;
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < kLaneKeys; ++i) {
        v[i] = i < left && i >= hidden ? v[i] * sc_log2 : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int d = kRowLanes / 2; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const float m_new = fmaxf(m_run, mx);  // finite: a tile has at least one visible key
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < kLaneKeys; i += 2) {
        const float e0 = exp2f(v[i] - m_new), e1 = exp2f(v[i + 1] - m_new);  // masked keys: 2^-inf = 0
        sum += e0 + e1;
        *reinterpret_cast<uint32_t*>(s_p + row * kProbLd + lk + i) = pack_bf16x2(e0, e1);
      }
#pragma unroll
      for (int d = kRowLanes / 2; d > 0; d >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
      const float alpha = exp2f(m_run - m_new);
      l_run = l_run * alpha + sum;
      m_run = m_new;
      if (lk == 0) s_alpha[row] = alpha;
    }
    named_bar_sync(1, kThreads);
    {
      uint32_t pa[kM][4][4];
      float al[kM][2];
      bool moved = false;
#pragma unroll
      for (int m = 0; m < kM; ++m) {
#pragma unroll
        for (int h = 0; h < 4; ++h)
          ldm_x4(smem_u32(s_p) + (m * 16 + (lane & 15)) * kProbLd * 2 + h * 32 + (lane >> 4) * 16, pa[m][h][0], pa[m][h][1], pa[m][h][2], pa[m][h][3]);
        al[m][0] = s_alpha[m * 16 + (lane >> 2)];
        al[m][1] = s_alpha[m * 16 + 8 + (lane >> 2)];
        moved = moved || al[m][0] != 1.f || al[m][1] != 1.f;
      }
      moved = __any_sync(0xffffffffu, moved);
#pragma unroll
      for (int a = 0; a < kPieces; ++a) {
        const int piece = warp + a * kWarps;
        if (piece >= out_pieces) break;
        if (a > 0) load_values(piece);
        if (moved) {
#pragma unroll
          for (int m = 0; m < kM; ++m)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
              o[a][m][j][0] *= al[m][0]; o[a][m][j][1] *= al[m][0];
              o[a][m][j][2] *= al[m][1]; o[a][m][j][3] *= al[m][1];
            }
        }
#pragma unroll
        for (int h = 0; h < 4; ++h)
#pragma unroll
          for (int m = 0; m < kM; ++m) {
            mma16816(o[a][m][0], pa[m][h], vb[h][0], vb[h][1]);
            mma16816(o[a][m][1], pa[m][h], vb[h][2], vb[h][3]);
          }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[st]);
    if (++st == p.stages) {
      st = 0;
      phase ^= 1;
    }
  }
  if (lk == 0) {
    if (p.parts == 1 && p.sink != nullptr && row < heads) l_run += sink_term(p, h0 + row, m_run);
    s_m[row] = m_run;
    s_l[row] = l_run;
  }
  named_bar_sync(1, kThreads);
  if (p.parts > 1 && threadIdx.x < heads) {
    float* ml = p.part_ml + ((static_cast<long long>(t) * p.H + h0 + threadIdx.x) * p.parts + part) * 2;
    ml[0] = s_m[threadIdx.x];
    ml[1] = s_l[threadIdx.x];
  }
#pragma unroll
  for (int a = 0; a < kPieces; ++a) {
    const int piece = warp + a * kWarps;
    if (piece >= out_pieces) break;
#pragma unroll
    for (int m = 0; m < kM; ++m)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = m * 16 + half * 8 + (lane >> 2);
        if (r >= heads) continue;
        const long long hrow = static_cast<long long>(t) * p.H + h0 + r;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int d = piece * 16 + j * 8 + (lane & 3) * 2;
          if (d >= p.rank) continue;  // the rank is a multiple of 8
          const float x = o[a][m][j][half * 2], y = o[a][m][j][half * 2 + 1];
          if (p.parts == 1) {
            const float l = s_l[r], inv = l > 0.f ? 1.f / l : 0.f;
            *reinterpret_cast<uint32_t*>(p.out + hrow * p.rank + d) = pack_bf16x2(x * inv, y * inv);
          } else {
            *reinterpret_cast<float2*>(p.part_o + (hrow * p.parts + part) * p.rank + d) = make_float2(x, y);
          }
        }
      }
  }
}

__global__ void __launch_bounds__(128) merge_kernel(Params p) {
  const int t = blockIdx.x, h = blockIdx.y;
  int seq = 0, ctx = 0;
  if (!locate(p, t, seq, ctx)) return;  // zeros are in place
  const int visible = ctx - (first_key(p, ctx) & ~(p.box - 1)), per = part_keys(p, visible);
  const int np = (visible + per - 1) / per;
  const long long hrow = static_cast<long long>(t) * p.H + h;
  const float* ml = p.part_ml + hrow * p.parts * 2;
  float m = -INFINITY, l = 0.f;
  for (int i = 0; i < np; ++i) m = fmaxf(m, ml[2 * i]);
  for (int i = 0; i < np; ++i) l += ml[2 * i + 1] * exp2f(ml[2 * i] - m);
  if (p.sink != nullptr) l += sink_term(p, h, m);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int d = threadIdx.x * 4; d < p.rank; d += 128 * 4) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int i = 0; i < np; ++i) {
      const float f = exp2f(ml[2 * i] - m) * inv;
      const float4 v = *reinterpret_cast<const float4*>(p.part_o + (hrow * p.parts + i) * p.rank + d);
      o.x = fmaf(v.x, f, o.x); o.y = fmaf(v.y, f, o.y); o.z = fmaf(v.z, f, o.z); o.w = fmaf(v.w, f, o.w);
    }
    *reinterpret_cast<uint2*>(p.out + hrow * p.rank + d) = make_uint2(pack_bf16x2(o.x, o.y), pack_bf16x2(o.z, o.w));
  }
}

template <int kM, int kPieces>
int launch(const CUtensorMap& tm, const Params& p, cudaStream_t s) {
  static bool attr_set = false;
  auto kern = paged_latent_kernel<kM, kPieces>;
  if (!attr_set) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem) != cudaSuccess) return kErrCuda;
    attr_set = true;
  }
  const int groups = (p.H + kM * 16 - 1) / (kM * 16);
  kern<<<dim3(p.T, groups, p.parts), cta_threads(kM, kPieces), smem_bytes(kM, p.width, p.stages), s>>>(tm, p);
  if (cudaGetLastError() != cudaSuccess) return kErrCuda;
  if (p.parts > 1) merge_kernel<<<dim3(p.T, p.H), 128, 0, s>>>(p);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

// ------------------------------------------------------------------------------------------------ per-head products
constexpr int kPT = 64, kPN = 64, kPK = 64;  // tile: rows, columns, inner
constexpr int kPLd = 72;                     // bf16 per staged row: an odd multiple of 16 bytes

struct ProductParams {
  const __nv_bfloat16 *a, *b;
  __nv_bfloat16* out;
  long long lda, a_head, ldb, b_head, ldo, o_head;
  int T, N, K;
  const __nv_bfloat16* gate;  // optional: the results of row t, head h are multiplied by the sigmoids of N numbers at gate + t * ldg + h * N
  long long ldg;
};

// kTrans: B(h) is [N, K] (out = A B^T), else [K, N]
template <bool kTrans>
__global__ void __launch_bounds__(128) head_product_kernel(ProductParams p) {
  __shared__ __align__(16) __nv_bfloat16 s_a[2][kPT * kPLd], s_b[2][64 * kPLd];
  const int n0 = blockIdx.x * kPN, t0 = blockIdx.y * kPT, h = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const __nv_bfloat16* A = p.a + h * p.a_head;
  const __nv_bfloat16* B = p.b + h * p.b_head;
  const int chunks = (p.K + kPK - 1) / kPK;
  // a [64 rows, 64 columns] tile of a matrix of `rows` x `cols`; what lies outside is zero
  auto copy = [&](__nv_bfloat16* dst, const __nv_bfloat16* src, long long ld, int r0, int rows, int c0, int cols) {
    for (int i = threadIdx.x; i < 64 * 8; i += 128) {
      const int r = i >> 3, c = (i & 7) * 8;
      __nv_bfloat16* d = dst + r * kPLd + c;
      if (r0 + r < rows && c0 + c < cols) cp16(d, src + (r0 + r) * ld + c0 + c);
      else *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
    }
  };
  auto issue = [&](int ch) {
    if (ch < chunks) {
      copy(s_a[ch & 1], A, p.lda, t0, p.T, ch * kPK, p.K);
      if constexpr (kTrans) copy(s_b[ch & 1], B, p.ldb, n0, p.N, ch * kPK, p.K);
      else copy(s_b[ch & 1], B, p.ldb, ch * kPK, p.K, n0, p.N);
    }
    cp_commit();
  };
  float acc[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j) { acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f; }
  issue(0);
  for (int ch = 0; ch < chunks; ++ch) {
    issue(ch + 1);
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const uint32_t sa = smem_u32(s_a[ch & 1]) + (warp * 16 + (lane & 15)) * kPLd * 2 + (lane >> 4) * 16;
    const uint32_t sb = smem_u32(s_b[ch & 1]);
#pragma unroll
    for (int ks = 0; ks < kPK / 16; ++ks) {
      uint32_t a[4];
      ldm_x4(sa + ks * 32, a[0], a[1], a[2], a[3]);
#pragma unroll
      for (int j = 0; j < 4; ++j) {  // pairs of 8-column tiles
        uint32_t b0, b1, b2, b3;
        if constexpr (kTrans) {
          // rows are columns of the result: (n 0-7, k 0-7), (n 0-7, k 8-15), (n 8-15, k 0-7), (n 8-15, k 8-15)
          ldm_x4(sb + (j * 16 + (lane >> 4) * 8 + (lane & 7)) * kPLd * 2 + ks * 32 + ((lane >> 3) & 1) * 16, b0, b1, b2, b3);
        } else {
          // (k 0-7, n 0-7), (k 8-15, n 0-7), (k 0-7, n 8-15), (k 8-15, n 8-15)
          ldm_x4_trans(sb + (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * kPLd * 2 + j * 32 + (lane >> 4) * 16, b0, b1, b2, b3);
        }
        mma16816(acc[2 * j], a, b0, b1);
        mma16816(acc[2 * j + 1], a, b2, b3);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int n = n0 + j * 8 + (lane & 3) * 2;
    if (n >= p.N) continue;  // N is a multiple of 8
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = t0 + warp * 16 + half * 8 + (lane >> 2);
      if (t >= p.T) continue;
      float a = acc[j][half * 2], b = acc[j][half * 2 + 1];
      if (p.gate != nullptr) {
        const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p.gate + t * p.ldg + h * p.N + n));
        a *= 1.f / (1.f + __expf(-g.x));
        b *= 1.f / (1.f + __expf(-g.y));
      }
      *reinterpret_cast<uint32_t*>(p.out + t * p.ldo + h * p.o_head + n) = pack_bf16x2(a, b);
    }
  }
}

}  // namespace latent
}  // namespace lvb

// Partitions of the visible keys that lvb_paged_latent uses for T rows of H heads: sizes part_o fp32 [T, H, parts, rank] and part_ml fp32 [T, H,
// parts, 2] (unused when 1).  The fewest waves of CTAs, set against the traffic of the merge: everything in units of the time that
// an SM takes to read a key.
extern "C" int lvb_paged_latent_parts(int T, int H, int width, int rank, int max_context, int window) {
  using namespace lvb;
  using namespace lvb::latent;
  if (T <= 0 || H <= 0 || width <= 0) return 1;
  const int keys = window > 0 && window < max_context ? window : max_context;
  const int m_tiles = H <= 16 ? 1 : 2, groups = (H + m_tiles * 16 - 1) / (m_tiles * 16);
  const int slots = num_sms();
  const double merge = 8.0 * T * H * rank / (2.0 * width * num_sms());
  int best = 1;
  double least = 0.;
  for (int parts = 1; parts <= 32 && (parts == 1 || keys / parts >= kMinPart); ++parts) {
    const long long ctas = static_cast<long long>(T) * groups * parts;
    const double cost = static_cast<double>((ctas + slots - 1) / slots) * (static_cast<double>(keys) / parts + kTileKeys) + (parts > 1 ? merge * parts + 64 : 0.);
    if (parts == 1 || cost < least) {
      least = cost;
      best = parts;
    }
  }
  return best;
}

// Packed query rows q [T, H, width] over pages [num_pages, page_size, width] whose rows' first `rank` elements are the values -> out [T, H, rank];
// causal, window > 0: a row sees itself and the window - 1 positions before it; sink (optional, fp32 [H]): joins the softmax denominator of its
// head, unscaled.  width and rank: multiples of 8, rank <= 512, width <= 576.
extern "C" int lvb_paged_latent(const void* q, const void* kv_pages, const int* kv_lens, const int* page_indices, const int* cu_q_lens,
                                const int* num_seqs, const float* sink, void* out, float* part_o, float* part_ml, int T, int H, int width,
                                int rank, int S, int pages_per_seq, int page_size, int num_pages, int window, int parts, float scale,
                                int* status, void* stream) {
  using namespace lvb;
  using namespace lvb::latent;
  if (T <= 0) return kErrOk;
  if (H <= 0 || width <= 0 || rank <= 0 || rank > width || ((width | rank) & 7) || S <= 0 || window < 0 || parts < 1) return kErrBadArg;
  if (rank > kMaxRank || width > 576) return kErrTooLarge;
  if (parts > 1 && (part_o == nullptr || part_ml == nullptr)) return kErrBadArg;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv_pages) | reinterpret_cast<uintptr_t>(out)) & 15) return kErrBadArg;
  Params p;
  p.q = reinterpret_cast<const __nv_bfloat16*>(q);
  p.kv_pages = reinterpret_cast<const __nv_bfloat16*>(kv_pages);
  p.kv_lens = kv_lens; p.page_indices = page_indices; p.cu_q_lens = cu_q_lens; p.num_seqs = num_seqs;
  p.sink = sink;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.part_o = part_o; p.part_ml = part_ml;
  p.T = T; p.H = H; p.width = width; p.rank = rank; p.S = S; p.pages_per_seq = pages_per_seq; p.page_size = page_size; p.num_pages = num_pages;
  p.parts = parts; p.window = window; p.scale = scale; p.status = status;
  const int m_tiles = H <= 16 ? 1 : 2;
  p.stages = kMaxStages;
  while (p.stages > 2 && smem_bytes(m_tiles, width, p.stages) > kMaxSmem) --p.stages;
  p.box = kTileKeys;
  p.box_log = 6;
  for (; page_size % p.box != 0; p.box /= 2) --p.box_log;
  CUtensorMap tm;
  // rows of an odd number of chunks are free of bank conflicts as they are; else the chunks are kept apart
  p.whole = (width & 63) == 0 && (chunks_of(width) & 1) != 0;
  p.grouped = (width & 63) == 0 && !p.whole;
  const uint64_t rows = static_cast<uint64_t>(num_pages) * page_size;
  const int rc = p.whole || p.grouped ? make_tmap_chunked_bf16(&tm, kv_pages, rows, width, p.box, p.grouped != 0)
                                      : make_tmap_2d_bf16(&tm, kv_pages, rows, width, width, p.box, 64);
  if (rc != kErrOk) return rc;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool narrow = rank <= 256;
  if (m_tiles == 1) return narrow ? launch<1, 2>(tm, p, s) : launch<1, 4>(tm, p, s);
  return narrow ? launch<2, 2>(tm, p, s) : launch<2, 4>(tm, p, s);
}

// out(t, h) [N] = A(t, h) [K] times B(h): [N, K] with b_trans, else [K, N].  A(t, h) starts at a + t * lda + h * a_head, B(h) at b + h * b_head (row
// stride ldb), out(t, h) at out + t * ldo + h * o_head.  bf16; N, K, lda, a_head, ldb, b_head multiples of 8, ldo, o_head and ldg of 2, a and b
// 16-byte aligned.  gate: null, or rows of H * N numbers (stride ldg, 4-byte aligned) whose sigmoids multiply the results.
extern "C" int lvb_head_product(const void* a, const void* b, void* out, const void* gate, int T, int H, int N, int K, long long lda,
                                long long a_head, long long ldb, long long b_head, long long ldo, long long o_head, long long ldg, int b_trans,
                                void* stream) {
  using namespace lvb;
  using namespace lvb::latent;
  if (T <= 0) return kErrOk;
  if (H <= 0 || N <= 0 || K <= 0 || ((N | K | lda | a_head | ldb | b_head) & 7) || ((ldo | o_head) & 1)) return kErrBadArg;
  if (((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(b)) & 15) || ((reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(gate)) & 3) || (ldg & 1))
    return kErrBadArg;
  if (H > 65535 || (T + kPT - 1) / kPT > 65535) return kErrTooLarge;
  ProductParams p{reinterpret_cast<const __nv_bfloat16*>(a), reinterpret_cast<const __nv_bfloat16*>(b), reinterpret_cast<__nv_bfloat16*>(out),
                  lda, a_head, ldb, b_head, ldo, o_head, T, N, K, reinterpret_cast<const __nv_bfloat16*>(gate), ldg};
  const dim3 grid((N + kPN - 1) / kPN, (T + kPT - 1) / kPT, H);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (b_trans) head_product_kernel<true><<<grid, 128, 0, s>>>(p);
  else head_product_kernel<false><<<grid, 128, 0, s>>>(p);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}
