// Latent attention over a paged cache, in the form in which every query head reads the same row per key: the row [c, k] of a key holds a
// compressed part c (rank elements) and a key part k shared by the heads, the query of head h is [W_uk(h)^T q, q'], the score is
// the product of the two rows, and the value is c itself (the caller applies W_uv(h) to the result).  So a key is read once for
// all heads and used twice.
//
//  * paged_latent: one CTA per (packed query row, group of up to 32 query heads, partition of the visible keys).  Keys arrive in
//    tiles of 32 rows by cp.async, several tiles deep.  Scores are warp-level MMAs (m16n8k16, bf16, fp32 accumulation) with the query
//    heads as the M rows; each warp takes 8 keys of one M tile (or, with 16 heads, 8 keys and half of the row), then owns the online
//    softmax of a few heads, and finally a set of 16-column pieces of the output, with the value operand read from the key tile by
//    transposing ldmatrix.  The visible keys of a row are cut evenly over the partitions inside the kernel, so the launch needs
//    no lengths from the device; a second kernel merges the partitions.
//  * head_product: out(t, h) = A(t, h) B(h) or A(t, h) B(h)^T for every head: the two products with per-head weights around it.
#include "common.cuh"

namespace lvb {
namespace latent {

constexpr int kThreads = 256;
constexpr int kTileKeys = 32;
constexpr int kMinPart = 64;   // keys of a partition, at least
constexpr int kMaxPieces = 4;  // 16-column output pieces per warp: rank <= 4 * 8 * 16
constexpr int kScoreLd = 36;   // floats per row of the score tile
constexpr int kProbLd = 40;    // bf16 per row of the probability tile

__device__ __forceinline__ void cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void ldm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldm_x2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
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
  __nv_bfloat16* out;             // [T, H, rank]
  float* part_o;                  // [T, H, parts, rank]
  float* part_ml;                 // [T, H, parts, 2]: maximum (base 2) and sum
  int T, H, width, rank, S, pages_per_seq, page_size, num_pages, parts, window, stages;
  float scale;
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

__host__ __device__ constexpr int row_bytes(int width) { return (width + 15) / 16 * 32 + 16; }  // an odd multiple of 16 bytes
__host__ __device__ constexpr int smem_bytes(int m_tiles, int width, int stages) {
  return (m_tiles * 16 + stages * kTileKeys) * row_bytes(width) + 32 * kScoreLd * 4 + m_tiles * 16 * kProbLd * 2 + m_tiles * 16 * 3 * 4 + 16;
}

// kM: M tiles (16 query heads each) per CTA
template <int kM>
__global__ void __launch_bounds__(kThreads, kM == 1 ? 2 : 1) paged_latent_kernel(Params p) {
  constexpr int kHeads = kM * 16;
  extern __shared__ __align__(16) uint8_t smem[];
  const int w16 = (p.width + 15) & ~15, rowb = row_bytes(p.width);
  uint8_t* s_q = smem;                                              // [kHeads][row]
  uint8_t* s_k = s_q + kHeads * rowb;                               // [stages][32][row]
  float* s_s = reinterpret_cast<float*>(s_k + p.stages * kTileKeys * rowb);  // kM = 1: two halves of [16][kScoreLd]; kM = 2: [32][kScoreLd]
  __nv_bfloat16* s_p = reinterpret_cast<__nv_bfloat16*>(s_s + 32 * kScoreLd);  // [kHeads][kProbLd]
  float* s_alpha = reinterpret_cast<float*>(s_p + kHeads * kProbLd);  // [kHeads]
  float* s_m = s_alpha + kHeads;
  float* s_l = s_m + kHeads;
  const int t = blockIdx.x, h0 = blockIdx.y * kHeads, part = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int heads = min(kHeads, p.H - h0);

  int seq = 0, ctx = 0;
  const bool live = locate(p, t, seq, ctx);
  const int first = live ? first_key(p, ctx) : 0;
  const int per = live ? part_keys(p, ctx - first) : 0;
  const int k0 = first + part * per;
  if (!live || k0 >= ctx) {
    if (!live && part == 0) {
      for (int i = threadIdx.x; i < heads * p.rank; i += kThreads)
        p.out[(static_cast<long long>(t) * p.H + h0) * p.rank + i] = __float2bfloat16(0.f);
    }
    return;
  }
  const int nk = min(per, ctx - k0);
  const int tiles = (nk + kTileKeys - 1) / kTileKeys;
  const int pieces = p.width / 8;  // 16-byte pieces of a row

  // queries; rows beyond the heads and columns beyond the width are zeros, in the key tiles too (those columns are never copied to)
  for (int i = threadIdx.x; i < kHeads * (w16 / 8); i += kThreads) {
    const int r = i / (w16 / 8), c = i - r * (w16 / 8);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < heads && c < pieces) v = *reinterpret_cast<const uint4*>(p.q + (static_cast<long long>(t) * p.H + h0 + r) * p.width + c * 8);
    *reinterpret_cast<uint4*>(s_q + r * rowb + c * 16) = v;
  }
  if (w16 != p.width) {
    for (int r = threadIdx.x; r < p.stages * kTileKeys; r += kThreads) *reinterpret_cast<uint4*>(s_k + r * rowb + pieces * 16) = make_uint4(0u, 0u, 0u, 0u);
  }
  auto issue = [&](int tile) {
    if (tile < tiles) {
      uint8_t* dst = s_k + (tile % p.stages) * kTileKeys * rowb;
      for (int r = warp; r < kTileKeys; r += kThreads / 32) {
        const int i = tile * kTileKeys + r;
        long long slot = -1;
        if (i < nk) {
          const int key = k0 + i;
          const int page = p.page_indices[seq * p.pages_per_seq + key / p.page_size];
          if (page >= 0 && page < p.num_pages) slot = static_cast<long long>(page) * p.page_size + key % p.page_size;
        }
        uint8_t* d = dst + r * rowb;
        if (slot >= 0) {
          const __nv_bfloat16* src = p.kv_pages + slot * p.width;
          for (int c = lane; c < pieces; c += 32) cp16(d + c * 16, src + c * 8);
        } else {
          for (int c = lane; c < pieces; c += 32) *reinterpret_cast<uint4*>(d + c * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
      }
    }
    cp_commit();
  };
  for (int i = 0; i < p.stages - 1; ++i) issue(i);

  const float sc_log2 = p.scale * 1.4426950408889634f;
  const int ksteps = w16 / 16, out_pieces = (p.rank + 15) / 16;
  // this warp's part of the scores
  const int mt = kM == 2 ? (warp & 1) : 0;
  const int nt = kM == 2 ? (warp >> 1) : (warp & 3);
  const int ks_lo = kM == 2 ? 0 : (warp >> 2) * ((ksteps + 1) / 2);
  const int ks_hi = kM == 2 ? ksteps : min(ksteps, ((warp >> 2) + 1) * ((ksteps + 1) / 2));
  float* my_scores = s_s + (kM == 2 ? mt * 16 : (warp >> 2) * 16) * kScoreLd;
  float m_run[2 * kM], l_run[2 * kM];  // heads warp * 2 kM + i, the same value in every lane
#pragma unroll
  for (int i = 0; i < 2 * kM; ++i) { m_run[i] = -INFINITY; l_run[i] = 0.f; }
  float o[kMaxPieces][kM][2][4];
#pragma unroll
  for (int a = 0; a < kMaxPieces; ++a)
#pragma unroll
    for (int b = 0; b < kM; ++b)
#pragma unroll
      for (int c = 0; c < 4; ++c) { o[a][b][0][c] = 0.f; o[a][b][1][c] = 0.f; }

  for (int it = 0; it < tiles; ++it) {
    // all but the newest stages - 2 groups have landed: tile `it` is there
    if (p.stages == 2) asm volatile("cp.async.wait_group 0;" ::: "memory");
    else if (p.stages == 3) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else asm volatile("cp.async.wait_group 2;" ::: "memory");
    __syncthreads();  // for everyone; and everyone is done with the tile before, whose buffer the next copy takes
    issue(it + p.stages - 1);
    const uint32_t kb = smem_u32(s_k + (it % p.stages) * kTileKeys * rowb);
    {
      float acc[2][4];
#pragma unroll
      for (int c = 0; c < 4; ++c) { acc[0][c] = 0.f; acc[1][c] = 0.f; }
      const uint32_t qa = smem_u32(s_q) + (mt * 16 + (lane & 15)) * rowb + (lane >> 4) * 16;
      const uint32_t ka = kb + (nt * 8 + (lane & 7)) * rowb + ((lane >> 3) & 1) * 16;
#pragma unroll 4
      for (int ks = ks_lo; ks < ks_hi; ++ks) {
        uint32_t a[4], b0, b1;
        ldm_x4(qa + ks * 32, a[0], a[1], a[2], a[3]);
        ldm_x2(ka + ks * 32, b0, b1);
        if (ks & 1) mma16816(acc[1], a, b0, b1);
        else mma16816(acc[0], a, b0, b1);
      }
      float* d = my_scores + (lane >> 2) * kScoreLd + nt * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(d) = make_float2(acc[0][0] + acc[1][0], acc[0][1] + acc[1][1]);
      *reinterpret_cast<float2*>(d + 8 * kScoreLd) = make_float2(acc[0][2] + acc[1][2], acc[0][3] + acc[1][3]);
    }
    __syncthreads();
    {
      const bool valid = it * kTileKeys + lane < nk;
#pragma unroll
      for (int i = 0; i < 2 * kM; ++i) {
        const int r = warp * 2 * kM + i;
        float v = s_s[r * kScoreLd + lane];
        if constexpr (kM == 1) v += s_s[(16 + r) * kScoreLd + lane];
        v = valid ? v * sc_log2 : -INFINITY;
        const float m_new = fmaxf(m_run[i], warp_max(v));
        const float e = valid ? exp2f(v - m_new) : 0.f;
        const float alpha = m_run[i] == -INFINITY ? 0.f : exp2f(m_run[i] - m_new);
        l_run[i] = l_run[i] * alpha + warp_sum(e);
        m_run[i] = m_new;
        s_p[r * kProbLd + lane] = __float2bfloat16(e);
        if (lane == 0) s_alpha[r] = alpha;
      }
    }
    __syncthreads();
    {
      uint32_t pa[kM][2][4];
      float al[kM][2];
#pragma unroll
      for (int m = 0; m < kM; ++m) {
#pragma unroll
        for (int h = 0; h < 2; ++h)
          ldm_x4(smem_u32(s_p) + (m * 16 + (lane & 15)) * kProbLd * 2 + h * 32 + (lane >> 4) * 16, pa[m][h][0], pa[m][h][1], pa[m][h][2], pa[m][h][3]);
        al[m][0] = s_alpha[m * 16 + (lane >> 2)];
        al[m][1] = s_alpha[m * 16 + 8 + (lane >> 2)];
      }
      // matrices of a transposing x4: (keys 0-7, columns 0-7), (keys 8-15, same), (keys 0-7, columns 8-15), (keys 8-15, same)
      const uint32_t va = kb + (((lane >> 3) & 1) * 8 + (lane & 7)) * rowb + (lane >> 4) * 16;
#pragma unroll
      for (int a = 0; a < kMaxPieces; ++a) {
        const int piece = warp + a * (kThreads / 32);
        if (piece >= out_pieces) break;
#pragma unroll
        for (int m = 0; m < kM; ++m)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            o[a][m][j][0] *= al[m][0]; o[a][m][j][1] *= al[m][0];
            o[a][m][j][2] *= al[m][1]; o[a][m][j][3] *= al[m][1];
          }
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          uint32_t b0, b1, b2, b3;
          ldm_x4_trans(va + h * 16 * rowb + piece * 32, b0, b1, b2, b3);
#pragma unroll
          for (int m = 0; m < kM; ++m) {
            mma16816(o[a][m][0], pa[m][h], b0, b1);
            mma16816(o[a][m][1], pa[m][h], b2, b3);
          }
        }
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < 2 * kM; ++i) {
      s_m[warp * 2 * kM + i] = m_run[i];
      s_l[warp * 2 * kM + i] = l_run[i];
    }
  }
  __syncthreads();
  if (p.parts > 1 && threadIdx.x < heads) {
    float* ml = p.part_ml + ((static_cast<long long>(t) * p.H + h0 + threadIdx.x) * p.parts + part) * 2;
    ml[0] = s_m[threadIdx.x];
    ml[1] = s_l[threadIdx.x];
  }
#pragma unroll
  for (int a = 0; a < kMaxPieces; ++a) {
    const int piece = warp + a * (kThreads / 32);
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
  const int visible = ctx - first_key(p, ctx), per = part_keys(p, visible);
  const int np = (visible + per - 1) / per;
  const long long hrow = static_cast<long long>(t) * p.H + h;
  const float* ml = p.part_ml + hrow * p.parts * 2;
  float m = -INFINITY, l = 0.f;
  for (int i = 0; i < np; ++i) m = fmaxf(m, ml[2 * i]);
  for (int i = 0; i < np; ++i) l += ml[2 * i + 1] * exp2f(ml[2 * i] - m);
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

template <int kM>
int launch(const Params& p, cudaStream_t s) {
  static bool attr_set = false;
  auto kern = paged_latent_kernel<kM>;
  if (!attr_set) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess) return kErrCuda;
    attr_set = true;
  }
  const int groups = (p.H + kM * 16 - 1) / (kM * 16);
  kern<<<dim3(p.T, groups, p.parts), kThreads, smem_bytes(kM, p.width, p.stages), s>>>(p);
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
      if (t < p.T) *reinterpret_cast<uint32_t*>(p.out + t * p.ldo + h * p.o_head + n) = pack_bf16x2(acc[j][half * 2], acc[j][half * 2 + 1]);
    }
  }
}

}  // namespace latent
}  // namespace lvb

// Partitions of the visible keys that lvb_paged_latent uses for T rows of H heads: sizes part_o fp32 [T, H, parts, rank] and part_ml fp32 [T, H,
// parts, 2] (unused when 1).
extern "C" int lvb_paged_latent_parts(int T, int H, int max_context, int window) {
  using namespace lvb;
  using namespace lvb::latent;
  const int keys = window > 0 && window < max_context ? window : max_context;
  const int groups = H <= 16 ? 1 : (H + 31) / 32;
  const int want = (2 * num_sms() + T * groups - 1) / (T * groups), most = (keys + 2 * kMinPart - 1) / (2 * kMinPart);
  const int parts = want < most ? want : most;
  return parts < 1 ? 1 : parts > 32 ? 32 : parts;
}

// Packed query rows q [T, H, width] over pages [num_pages, page_size, width] whose rows' first `rank` elements are the values -> out [T, H, rank];
// causal, window > 0: a row sees itself and the window - 1 positions before it.  width and rank: multiples of 8, rank <= 512, width <= 640.
extern "C" int lvb_paged_latent(const void* q, const void* kv_pages, const int* kv_lens, const int* page_indices, const int* cu_q_lens,
                                const int* num_seqs, void* out, float* part_o, float* part_ml, int T, int H, int width, int rank, int S,
                                int pages_per_seq, int page_size, int num_pages, int window, int parts, float scale, void* stream) {
  using namespace lvb;
  using namespace lvb::latent;
  if (T <= 0) return kErrOk;
  if (H <= 0 || width <= 0 || rank <= 0 || rank > width || ((width | rank) & 7) || S <= 0 || window < 0 || parts < 1) return kErrBadArg;
  if (rank > kMaxPieces * 8 * 16 || width > 640) return kErrTooLarge;
  if (parts > 1 && (part_o == nullptr || part_ml == nullptr)) return kErrBadArg;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv_pages) | reinterpret_cast<uintptr_t>(out)) & 15) return kErrBadArg;
  Params p;
  p.q = reinterpret_cast<const __nv_bfloat16*>(q);
  p.kv_pages = reinterpret_cast<const __nv_bfloat16*>(kv_pages);
  p.kv_lens = kv_lens; p.page_indices = page_indices; p.cu_q_lens = cu_q_lens; p.num_seqs = num_seqs;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.part_o = part_o; p.part_ml = part_ml;
  p.T = T; p.H = H; p.width = width; p.rank = rank; p.S = S; p.pages_per_seq = pages_per_seq; p.page_size = page_size; p.num_pages = num_pages;
  p.parts = parts; p.window = window; p.scale = scale;
  const int m_tiles = H <= 16 ? 1 : 2;
  const int room = (m_tiles == 1 ? 110 : 216) * 1024;
  p.stages = 4;
  while (p.stages > 2 && smem_bytes(m_tiles, width, p.stages) > room) --p.stages;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return m_tiles == 1 ? launch<1>(p, s) : launch<2>(p, s);
}

// out(t, h) [N] = A(t, h) [K] times B(h): [N, K] with b_trans, else [K, N].  A(t, h) starts at a + t * lda + h * a_head, B(h) at b + h * b_head (row
// stride ldb), out(t, h) at out + t * ldo + h * o_head.  bf16; N, K, lda, a_head, ldb, b_head multiples of 8, ldo and o_head of 2, a and b
// 16-byte aligned.
extern "C" int lvb_head_product(const void* a, const void* b, void* out, int T, int H, int N, int K, long long lda, long long a_head, long long ldb,
                                long long b_head, long long ldo, long long o_head, int b_trans, void* stream) {
  using namespace lvb;
  using namespace lvb::latent;
  if (T <= 0) return kErrOk;
  if (H <= 0 || N <= 0 || K <= 0 || ((N | K | lda | a_head | ldb | b_head) & 7) || ((ldo | o_head) & 1)) return kErrBadArg;
  if (((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(b)) & 15) || (reinterpret_cast<uintptr_t>(out) & 3)) return kErrBadArg;
  if (H > 65535 || (T + kPT - 1) / kPT > 65535) return kErrTooLarge;
  ProductParams p{reinterpret_cast<const __nv_bfloat16*>(a), reinterpret_cast<const __nv_bfloat16*>(b), reinterpret_cast<__nv_bfloat16*>(out),
                  lda, a_head, ldb, b_head, ldo, o_head, T, N, K};
  const dim3 grid((N + kPN - 1) / kPN, (T + kPT - 1) / kPT, H);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (b_trans) head_product_kernel<true><<<grid, 128, 0, s>>>(p);
  else head_product_kernel<false><<<grid, 128, 0, s>>>(p);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}
