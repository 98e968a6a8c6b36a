// Linear attention with a fixed decay per head over packed rows, with a matrix state per sequence slot:
//   S_t = decay S_{t-1} + (key_scale k_t) v_t^T,   o_t = S_t^T q_t        (S [dk, dv] fp32 per head),
// and the norm of its outputs in groups times an activated gate.  Sequence boundaries, lengths and slots are read from device arrays.
// The state, decays and everything added to the state are 32-bit; this file is built without fast-math.
//
// Decode rounds (and fp32, and sizes that are not multiples of 8) walk a sequence row by row with 32 columns of a head's state in
// registers.  Prompts in bf16 are cut into pieces of chunks.  A first kernel sums up what every piece but a sequence's last adds to the
// state, a second one turns these sums into the states that the pieces start from, and the third walks all pieces at once on the
// tensor cores: with D the decays between the rows of a chunk,
//   O = decay^(i+1) (Q S) + ((Q K^T) o D) V,   S <- decay^n S + (K o decay^(n-1-j))^T V.
// The fp32 state stays in accumulators; the products that read it, and the decayed factor that enters it, use two bf16 parts per number,
// so that what is rounded to 16 bits is only what came in 16 bits, and the weights (Q K^T) o D as in the other attentions.
// Keys of up to 128 run on tcgen05 (linear_attention_umma.cu); keys of up to 256, whose tiles leave no room for that, on warp-level MMAs
// (below).
#include "linear_attention.cuh"
#include "row_groups.cuh"

namespace lvb {
namespace linattn {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void store1(float* p, float v) { *p = v; }
__device__ __forceinline__ void store1(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// ------------------------------------------------------------------------------------------------ row by row
constexpr int kCols = 32;  // columns of a head's state per CTA
constexpr int kStepThreads = 256;
constexpr int kStepRows = kStepThreads / (kCols / 4);  // rows of the state side by side

// kQ: rows of the state per thread, dk <= kQ * 32.  A thread holds 4 columns of each.
template <typename T, int kQ>
__global__ void __launch_bounds__(kStepThreads) step_kernel(Params p) {
  __shared__ float s_q[kQ * kStepRows], s_k[kQ * kStepRows], s_v[kCols];
  __shared__ float s_o[kStepThreads / 32][kCols];
  const int h = blockIdx.y, c0 = blockIdx.x * kCols;
  const int n_seq = live_sequences(p);
  T* out = reinterpret_cast<T*>(p.out) + h * p.dv + c0;
  const long long ldo = static_cast<long long>(p.H) * p.dv;
  if (static_cast<int>(blockIdx.z) == p.S) {  // rows of no sequence: zeros
    const int c = threadIdx.x & 31;
    for (int r = (n_seq > 0 ? p.cu_q_lens[n_seq] : 0) + (threadIdx.x >> 5); r < p.T; r += kStepThreads / 32)
      if (c0 + c < p.dv) store1(out + r * ldo + c, 0.f);
    return;
  }
  Sequence s;
  if (static_cast<int>(blockIdx.z) >= n_seq || !sequence(p, blockIdx.z, s)) return;
  const int col = (threadIdx.x & 7) * 4, row = threadIdx.x >> 3, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const bool vec = (p.dv & 3) == 0;
  float* st = p.state + (static_cast<long long>(s.slot) * p.H + h) * p.dk * p.dv + c0 + col;
  const int cols = min(max(p.dv - c0 - col, 0), 4);
  float a[kQ][4];
#pragma unroll
  for (int j = 0; j < kQ; ++j) {
    const int d = row + j * kStepRows;
    a[j][0] = a[j][1] = a[j][2] = a[j][3] = 0.f;
    if (!s.from_state || d >= p.dk) continue;
    const float* src = st + static_cast<long long>(d) * p.dv;
    if (vec && cols == 4) {
      const float4 x = *reinterpret_cast<const float4*>(src);
      a[j][0] = x.x; a[j][1] = x.y; a[j][2] = x.z; a[j][3] = x.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (e < cols) a[j][e] = src[e];
    }
  }
  const float g = p.decay[h];
  auto in = [&](const void* base, long long i) {
    const float x = to_f(reinterpret_cast<const T*>(base)[i]);
    return p.silu ? x / (1.f + expf(-x)) : x;
  };
  for (int r = s.r0; r < s.r1; ++r) {
    const long long at = r * p.ld + h * p.dk;
    for (int e = threadIdx.x; e < kQ * kStepRows; e += kStepThreads) {
      s_q[e] = e < p.dk ? in(p.q, at + e) : 0.f;
      s_k[e] = e < p.dk ? in(p.k, at + e) * p.key_scale : 0.f;
    }
    if (threadIdx.x < kCols) s_v[threadIdx.x] = c0 + threadIdx.x < p.dv ? in(p.v, r * p.ld + h * p.dv + c0 + threadIdx.x) : 0.f;
    __syncthreads();
    float v[4], o[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) { v[e] = s_v[col + e]; o[e] = 0.f; }
#pragma unroll
    for (int j = 0; j < kQ; ++j) {
      const float kd = s_k[row + j * kStepRows], qd = s_q[row + j * kStepRows];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        a[j][e] = fmaf(g, a[j][e], kd * v[e]);
        o[e] = fmaf(qd, a[j][e], o[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      o[e] += __shfl_xor_sync(0xffffffffu, o[e], 8);
      o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
    }
    if (lane < 8) *reinterpret_cast<float4*>(&s_o[warp][col]) = make_float4(o[0], o[1], o[2], o[3]);
    __syncthreads();  // also: this row's q, k and v have been read
    if (threadIdx.x < kCols && c0 + threadIdx.x < p.dv) {
      float t = 0.f;
#pragma unroll
      for (int w = 0; w < kStepThreads / 32; ++w) t += s_o[w][threadIdx.x];
      store1(out + r * ldo + threadIdx.x, t);
    }
  }
#pragma unroll
  for (int j = 0; j < kQ; ++j) {
    const int d = row + j * kStepRows;
    if (d >= p.dk) continue;
    float* dst = st + static_cast<long long>(d) * p.dv;
    if (vec && cols == 4) *reinterpret_cast<float4*>(dst) = make_float4(a[j][0], a[j][1], a[j][2], a[j][3]);
    else
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (e < cols) dst[e] = a[j][e];
  }
}

// ------------------------------------------------------------------------------------------------ by chunks
constexpr int kC = 64;  // rows of a chunk
constexpr int kChunkThreads = 128;

__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool in) {  // zeros when !in
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int kLeft> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(kLeft) : "memory"); }
__device__ __forceinline__ void ldm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldm_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Byte offset of 16-byte unit u of row r in a tile with rows of kBytes; eight consecutive rows' units u fall into eight different
// bank groups.
template <int kBytes>
__device__ __forceinline__ uint32_t unit_at(int r, int u) {
  if constexpr (kBytes >= 128) return r * kBytes + ((u ^ (r & 7)) << 4);
  else return r * kBytes + ((u ^ ((r >> 1) & 3)) << 4);
}

template <int kDK, int kDV>
struct Tiles {
  static constexpr int kQBytes = kDK * 2, kVBytes = kDV * 2;  // of a row
  static constexpr int kStage = kC * (2 * kQBytes + kVBytes); // q, k, v
  static constexpr int kStateAt = 2 * kStage;
  static constexpr int kSmem = kStateAt + 2 * kDK * kVBytes;  // the state in two parts
  // warps over the state: kMW along dk, kNW along dv
  static constexpr int kMW = kDK >= 64 ? 4 : 2, kNW = 4 / kMW;
  static constexpr int kMT = kDK / kMW / 16, kNT = kDV / kNW / 8;
};

// kStateOnly: what a piece adds to a zero state, for all pieces but the last of a sequence.  Otherwise: the outputs of every piece, and the
// state after a sequence's last.
template <int kDK, int kDV, bool kStateOnly>
__global__ void __launch_bounds__(kChunkThreads, 2) chunk_kernel(Params p) {
  using Tl = Tiles<kDK, kDV>;
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float s_pow[kC + 1];
  const int h = blockIdx.y, c0 = blockIdx.z * kDV;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const long long ldo = static_cast<long long>(p.H) * p.dv;
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + h * p.dv + c0;
  int seq = 0, c = 0, of = 0;
  if (!find_piece(p, blockIdx.x, seq, c, of)) {
    if constexpr (!kStateOnly) {  // the work items past the last piece (there is always one): zeros for the rows of no sequence
      const int n_seq = live_sequences(p);
      const int cols = min(p.dv - c0, kDV);
      for (int r = (n_seq > 0 ? p.cu_q_lens[n_seq] : 0) + blockIdx.x - of; r < p.T; r += gridDim.x - of)
        for (int e = tid; e < cols; e += kChunkThreads) out[r * ldo + e] = __float2bfloat16(0.f);
    }
    return;
  }
  Sequence s;
  if (!sequence(p, seq, s)) return;
  if (kStateOnly && c == of - 1) return;
  const int r0 = s.r0 + c * p.piece, rows = min(p.piece, s.r1 - r0), chunks = (rows + kC - 1) / kC;
  const float decay = p.decay[h];
  if (tid <= kC) s_pow[tid] = powf(decay, static_cast<float>(tid));
  const uint32_t base = smem_u32(smem);
  const long long head = static_cast<long long>(p.dk) * p.dv;
  const float* from = nullptr;
  if constexpr (!kStateOnly) {
    if (of > 1) from = p.pieces + (static_cast<long long>(blockIdx.x) * p.H + h) * head + c0;
    else if (s.from_state) from = p.state + (static_cast<long long>(s.slot) * p.H + h) * head + c0;
  }
  const int wm = (warp % Tl::kMW) * (kDK / Tl::kMW), wn = (warp / Tl::kMW) * (kDV / Tl::kNW);
  const int fr = lane >> 2, fc = (lane & 3) * 2;  // row and columns of a fragment's first pair
  // this warp's part of the state: rows wm + mt * 16 + fr (+ 8), columns wn + nt * 8 + fc (+ 1)
  float st[Tl::kMT][Tl::kNT][4];
#pragma unroll
  for (int mt = 0; mt < Tl::kMT; ++mt)
#pragma unroll
    for (int nt = 0; nt < Tl::kNT; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = wm + mt * 16 + fr + e * 8, cc = wn + nt * 8 + fc;
        float2 x = make_float2(0.f, 0.f);
        if (from != nullptr && d < p.dk && c0 + cc < p.dv) x = *reinterpret_cast<const float2*>(from + static_cast<long long>(d) * p.dv + cc);
        st[mt][nt][2 * e] = x.x;
        st[mt][nt][2 * e + 1] = x.y;
      }
  auto leave_state = [&] {  // as two bf16 parts, for the products that read it
#pragma unroll
    for (int mt = 0; mt < Tl::kMT; ++mt)
#pragma unroll
      for (int nt = 0; nt < Tl::kNT; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          uint32_t hi, lo;
          split2(st[mt][nt][2 * e], st[mt][nt][2 * e + 1], hi, lo);
          uint8_t* dst = smem + Tl::kStateAt + unit_at<Tl::kVBytes>(wm + mt * 16 + fr + e * 8, (wn >> 3) + nt) + fc * 2;
          *reinterpret_cast<uint32_t*>(dst) = hi;
          *reinterpret_cast<uint32_t*>(dst + kDK * Tl::kVBytes) = lo;
        }
  };
  if constexpr (!kStateOnly) leave_state();
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.q) + h * p.dk;
  const __nv_bfloat16* k = reinterpret_cast<const __nv_bfloat16*>(p.k) + h * p.dk;
  const __nv_bfloat16* v = reinterpret_cast<const __nv_bfloat16*>(p.v) + h * p.dv + c0;
  auto issue = [&](int ch) {
    if (ch < chunks) {
      const uint32_t at = base + (ch & 1) * Tl::kStage;
      const int n = rows - ch * kC;
      const long long first = static_cast<long long>(r0 + ch * kC) * p.ld;
      for (int i = tid; i < kC * (kDK / 8); i += kChunkThreads) {
        const int r = i / (kDK / 8), u = i % (kDK / 8);
        const bool in = r < n && u * 8 < p.dk;
        const long long src = in ? first + r * p.ld + u * 8 : first;
        if constexpr (!kStateOnly) cp16(at + unit_at<Tl::kQBytes>(r, u), q + src, in);
        cp16(at + kC * Tl::kQBytes + unit_at<Tl::kQBytes>(r, u), k + src, in);
      }
      for (int i = tid; i < kC * (kDV / 8); i += kChunkThreads) {
        const int r = i / (kDV / 8), u = i % (kDV / 8);
        const bool in = r < n && c0 + u * 8 < p.dv;
        cp16(at + 2 * kC * Tl::kQBytes + unit_at<Tl::kVBytes>(r, u), in ? v + first + r * p.ld + u * 8 : v, in);
      }
    }
    cp_commit();
  };
  issue(0);
  for (int ch = 0; ch < chunks; ++ch) {
    issue(ch + 1);
    cp_wait<1>();
    __syncthreads();  // the chunk has arrived, and so has the state
    const uint32_t sq = base + (ch & 1) * Tl::kStage, sk = sq + kC * Tl::kQBytes, sv = sk + kC * Tl::kQBytes, ss = base + Tl::kStateAt;
    const int n = min(rows - ch * kC, kC);
    if constexpr (!kStateOnly) {
      // rows warp * 16 .. + 15 of the chunk: scores with the rows up to them, what the state gives, what the chunk gives
      const int blocks = warp + 1;  // blocks of 16 keys
      float o[kDV / 8][4];
#pragma unroll
      for (int j = 0; j < kDV / 8; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
      float sc[kC / 8][4];
#pragma unroll
      for (int j = 0; j < kC / 8; ++j) { sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f; }
#pragma unroll
      for (int ks = 0; ks < kDK / 16; ++ks) {
        uint32_t a[4];
        ldm_x4(sq + unit_at<Tl::kQBytes>(warp * 16 + (lane & 15), ks * 2 + (lane >> 4)), a);
#pragma unroll
        for (int j = 0; j < kDV / 16; ++j) {
          const uint32_t at = unit_at<Tl::kVBytes>(ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), j * 2 + (lane >> 4));
          uint32_t b[4];
          ldm_x4_trans(ss + at, b);
          mma16816(o[2 * j], a, b[0], b[1]);
          mma16816(o[2 * j + 1], a, b[2], b[3]);
          ldm_x4_trans(ss + kDK * Tl::kVBytes + at, b);
          mma16816(o[2 * j], a, b[0], b[1]);
          mma16816(o[2 * j + 1], a, b[2], b[3]);
        }
#pragma unroll
        for (int j = 0; j < kC / 16; ++j) {
          if (j >= blocks) continue;
          uint32_t b[4];
          ldm_x4(sk + unit_at<Tl::kQBytes>(j * 16 + (lane >> 4) * 8 + (lane & 7), ks * 2 + ((lane >> 3) & 1)), b);
          mma16816(sc[2 * j], a, b[0], b[1]);
          mma16816(sc[2 * j + 1], a, b[2], b[3]);
        }
      }
      const int i0 = warp * 16 + fr;
      const float p0 = s_pow[i0 + 1], p1 = s_pow[i0 + 9];
#pragma unroll
      for (int j = 0; j < kDV / 8; ++j) { o[j][0] *= p0; o[j][1] *= p0; o[j][2] *= p1; o[j][3] *= p1; }
#pragma unroll
      for (int j = 0; j < kC / 16; ++j) {
        if (j >= blocks) continue;
        uint32_t a[4];
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          float x[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int back = i0 + (e >> 1) * 8 - (j * 16 + t * 8 + fc + (e & 1));
            x[e] = back >= 0 ? sc[2 * j + t][e] * (s_pow[back] * p.key_scale) : 0.f;
          }
          a[2 * t] = pack_bf16x2(x[0], x[1]);
          a[2 * t + 1] = pack_bf16x2(x[2], x[3]);
        }
#pragma unroll
        for (int jn = 0; jn < kDV / 16; ++jn) {
          uint32_t b[4];
          ldm_x4_trans(sv + unit_at<Tl::kVBytes>(j * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), jn * 2 + (lane >> 4)), b);
          mma16816(o[2 * jn], a, b[0], b[1]);
          mma16816(o[2 * jn + 1], a, b[2], b[3]);
        }
      }
      __nv_bfloat16* to = out + static_cast<long long>(r0 + ch * kC) * ldo;
#pragma unroll
      for (int j = 0; j < kDV / 8; ++j) {
        if (c0 + j * 8 + fc >= p.dv) continue;
        if (i0 < n) *reinterpret_cast<uint32_t*>(to + i0 * ldo + j * 8 + fc) = pack_bf16x2(o[j][0], o[j][1]);
        if (i0 + 8 < n) *reinterpret_cast<uint32_t*>(to + (i0 + 8) * ldo + j * 8 + fc) = pack_bf16x2(o[j][2], o[j][3]);
      }
    }
    // S <- decay^n S + (K o decay^(n - 1 - j))^T V
    {
      const float dn = s_pow[n];
#pragma unroll
      for (int mt = 0; mt < Tl::kMT; ++mt)
#pragma unroll
        for (int nt = 0; nt < Tl::kNT; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) st[mt][nt][e] *= dn;
#pragma unroll
      for (int ks = 0; ks < kC / 16; ++ks) {
        if (ks * 16 >= n) continue;
        float f[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int left = n - 1 - (ks * 16 + (e >> 1) * 8 + fc + (e & 1));
          f[e] = left >= 0 ? s_pow[left] * p.key_scale : 0.f;
        }
        uint32_t hi[Tl::kMT][4], lo[Tl::kMT][4];
#pragma unroll
        for (int mt = 0; mt < Tl::kMT; ++mt) {
          uint32_t a[4];
          ldm_x4_trans(sk + unit_at<Tl::kQBytes>(ks * 16 + (lane >> 4) * 8 + (lane & 7), (wm >> 3) + mt * 2 + ((lane >> 3) & 1)), a);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a[e]));
            split2(x.x * f[(e >> 1) * 2], x.y * f[(e >> 1) * 2 + 1], hi[mt][e], lo[mt][e]);
          }
        }
#pragma unroll
        for (int j = 0; j < Tl::kNT / 2; ++j) {
          uint32_t b[4];
          ldm_x4_trans(sv + unit_at<Tl::kVBytes>(ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), (wn >> 3) + j * 2 + (lane >> 4)), b);
#pragma unroll
          for (int mt = 0; mt < Tl::kMT; ++mt) {
            mma16816(st[mt][2 * j], hi[mt], b[0], b[1]);
            mma16816(st[mt][2 * j + 1], hi[mt], b[2], b[3]);
            mma16816(st[mt][2 * j], lo[mt], b[0], b[1]);
            mma16816(st[mt][2 * j + 1], lo[mt], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();  // everyone is done with this chunk's tiles and with the state
    if constexpr (!kStateOnly) {
      if (ch + 1 < chunks) leave_state();
    }
  }
  cp_wait<0>();
  if (!kStateOnly && c != of - 1) return;
  float* to = kStateOnly ? p.pieces + (static_cast<long long>(blockIdx.x) * p.H + h) * head + c0
                         : p.state + (static_cast<long long>(s.slot) * p.H + h) * head + c0;
#pragma unroll
  for (int mt = 0; mt < Tl::kMT; ++mt)
#pragma unroll
    for (int nt = 0; nt < Tl::kNT; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = wm + mt * 16 + fr + e * 8, cc = wn + nt * 8 + fc;
        if (d < p.dk && c0 + cc < p.dv)
          *reinterpret_cast<float2*>(to + static_cast<long long>(d) * p.dv + cc) = make_float2(st[mt][nt][2 * e], st[mt][nt][2 * e + 1]);
      }
}

// pieces: what each piece adds -> the state that each piece starts from, for sequences of more than one piece.  dk * dv is a multiple of 4.
__global__ void __launch_bounds__(256) carry_kernel(Params p) {
  __shared__ int s_first, s_of;
  const int i = blockIdx.z, h = blockIdx.y;
  if (i >= live_sequences(p)) return;
  if (threadIdx.x == 0) s_first = 0;
  __syncthreads();
  int part = 0;
  for (int j = threadIdx.x; j < i; j += 256) part += (max(min(p.cu_q_lens[j + 1], p.T) - max(p.cu_q_lens[j], 0), 0) + p.piece - 1) / p.piece;
  if (part) atomicAdd(&s_first, part);
  Sequence s;
  const bool ok = sequence(p, i, s);
  if (threadIdx.x == 0) s_of = ok ? (s.r1 - s.r0 + p.piece - 1) / p.piece : 0;
  __syncthreads();
  const int first = s_first, of = s_of;
  const long long head = static_cast<long long>(p.dk) * p.dv, e = (static_cast<long long>(blockIdx.x) * 256 + threadIdx.x) * 4;
  if (of < 2 || e >= head) return;
  const float f = powf(p.decay[h], static_cast<float>(p.piece));
  float4 run = make_float4(0.f, 0.f, 0.f, 0.f);
  if (s.from_state) run = *reinterpret_cast<const float4*>(p.state + (static_cast<long long>(s.slot) * p.H + h) * head + e);
  float* at = p.pieces + (static_cast<long long>(first) * p.H + h) * head + e;
  const long long step = p.H * head;
  float4 next = *reinterpret_cast<const float4*>(at);
  for (int c = 0; c < of; ++c, at += step) {
    const float4 add = next;
    if (c + 2 < of) next = *reinterpret_cast<const float4*>(at + step);
    *reinterpret_cast<float4*>(at) = run;
    run.x = fmaf(f, run.x, add.x);
    run.y = fmaf(f, run.y, add.y);
    run.z = fmaf(f, run.z, add.z);
    run.w = fmaf(f, run.w, add.w);
  }
}

void carry_states(const Params& p, cudaStream_t s) {
  const long long head = static_cast<long long>(p.dk) * p.dv;
  carry_kernel<<<dim3(static_cast<unsigned>((head / 4 + 255) / 256), p.H, p.S), 256, 0, s>>>(p);
}

template <int kDK, int kDV>
int run_chunks(const Params& p, int items, cudaStream_t s) {
  using Tl = Tiles<kDK, kDV>;
  const dim3 grid(items, p.H, (p.dv + kDV - 1) / kDV);
  if (cudaFuncSetAttribute(chunk_kernel<kDK, kDV, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, Tl::kSmem) != cudaSuccess ||
      cudaFuncSetAttribute(chunk_kernel<kDK, kDV, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, Tl::kStateAt) != cudaSuccess)
    return kErrCuda;
  if (p.pieces != nullptr) {
    chunk_kernel<kDK, kDV, true><<<grid, kChunkThreads, Tl::kStateAt, s>>>(p);
    carry_states(p, s);
  }
  chunk_kernel<kDK, kDV, false><<<grid, kChunkThreads, Tl::kSmem, s>>>(p);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

template <typename T>
int run_steps(const Params& p, cudaStream_t s) {
  const dim3 grid((p.dv + kCols - 1) / kCols, p.H, p.S + 1);
  if (p.dk <= 32) step_kernel<T, 1><<<grid, kStepThreads, 0, s>>>(p);
  else if (p.dk <= 64) step_kernel<T, 2><<<grid, kStepThreads, 0, s>>>(p);
  else if (p.dk <= 128) step_kernel<T, 4><<<grid, kStepThreads, 0, s>>>(p);
  else if (p.dk <= 256) step_kernel<T, 8><<<grid, kStepThreads, 0, s>>>(p);
  else if (p.dk <= 512) step_kernel<T, 16><<<grid, kStepThreads, 0, s>>>(p);
  else return kErrTooLarge;
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}

// ------------------------------------------------------------------------------------------------ what follows the recurrence
// y[t] = o[t] with every group divided by its root mean square, times w (optional), times act(gate[t]): silu (0) or sigmoid (1)
template <int kN, int kVec, int kThreads>
__global__ void __launch_bounds__(kThreads)
gated_norm_kernel(const void* __restrict__ o, const void* __restrict__ gate, long long ldg, const void* __restrict__ w, int w_f32, void* __restrict__ y,
                  int f32, int dim, int part, float eps, int act) {
  using Row = rowg::Row<kN, kVec>;
  extern __shared__ float s_norm[];
  const size_t at = static_cast<size_t>(blockIdx.x) * dim;
  Row x;
  float g[kN][kVec];
#pragma unroll
  for (int n = 0; n < kN; ++n) {
#pragma unroll
    for (int e = 0; e < kVec; ++e) x.a[n][e] = 0.f;
    if (Row::column(n) >= dim) continue;
    rowg::ld_unit<kVec>(o, f32, at + Row::column(n), x.a[n]);
    rowg::ld_unit<kVec>(gate, f32, static_cast<size_t>(blockIdx.x) * ldg + Row::column(n), g[n]);
  }
  x.normalize(typename Row::Groups(dim, part), eps, s_norm);
#pragma unroll
  for (int n = 0; n < kN; ++n) {
    const int col = Row::column(n);
    if (col >= dim) continue;
    float m[kVec];
    if (w != nullptr) rowg::ld_unit<kVec>(w, w_f32, col, m);
#pragma unroll
    for (int e = 0; e < kVec; ++e) {
      // (a gate that multiplies 16-bit results needs no more than the fast forms)
      const float s = f32 ? 1.f / (1.f + expf(-g[n][e])) : __fdividef(1.f, 1.f + __expf(-g[n][e]));
      x.a[n][e] *= (act == 0 ? g[n][e] * s : s) * (w != nullptr ? m[e] : 1.f);
    }
    rowg::st_unit<kVec>(y, f32, at + col, x.a[n]);
  }
}

// Eight consecutive bf16 numbers.
struct Eight {
  float v[8];
  __device__ __forceinline__ void load(const void* p, long long i) {
    const uint4 w = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p) + i);
    const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u[e]));
      v[2 * e] = f.x;
      v[2 * e + 1] = f.y;
    }
  }
  __device__ __forceinline__ void store(void* p, long long i) const {
    *reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(p) + i) =
        make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
  }
  __device__ __forceinline__ float squares() const {
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) s = fmaf(v[e], v[e], s);
    return s;
  }
  // times r, w and act(gate)
  __device__ __forceinline__ void finish(float r, const Eight& gate, const void* w, int w_f32, int col, int act) {
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float s = __fdividef(1.f, 1.f + __expf(-gate.v[e]));
      v[e] *= r * (act == 0 ? gate.v[e] * s : s) * (w != nullptr ? rowg::ld1(w, w_f32, col + e) : 1.f);
    }
  }
};

// gated_norm_kernel for bf16 rows and groups of 8, 16, .. 256 elements: `lanes` neighbouring lanes hold a group, and no warp waits for another.
__global__ void __launch_bounds__(256)
gated_norm_small_kernel(const void* __restrict__ o, const void* __restrict__ gate, long long ldg, const void* __restrict__ w, int w_f32,
                        void* __restrict__ y, long long units, int per_row, int lanes, float eps, int act) {
  const float inv = 1.f / static_cast<float>(lanes * 8);
  const long long step = static_cast<long long>(gridDim.x) * 256;
  for (long long base = static_cast<long long>(blockIdx.x) * 256; base < units; base += step) {  // whole warps: the sums are made together
    const long long i = base + threadIdx.x;
    const bool in = i < units;
    const long long r = in ? i / per_row : 0;
    const int col = in ? static_cast<int>(i - r * per_row) * 8 : 0;
    Eight x, g;
    x.load(o, in ? i * 8 : 0);
    g.load(gate, r * ldg + col);
    float ss = x.squares();
    for (int m = 1; m < lanes; m <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
    x.finish(1.f / sqrtf(ss * inv + eps), g, w, w_f32, col, act);
    if (in) x.store(y, i * 8);
  }
}

// The same for one group per row; a CTA per row, kU units of 8 per thread.
template <int kU>
__global__ void __launch_bounds__(512)
gated_norm_row_kernel(const void* __restrict__ o, const void* __restrict__ gate, long long ldg, const void* __restrict__ w, int w_f32,
                      void* __restrict__ y, int dim, float eps, int act) {
  __shared__ float s_sum[16];
  const long long row = blockIdx.x;
  Eight x[kU], g[kU];
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < kU; ++u) {
    const int col = (threadIdx.x + u * blockDim.x) * 8;
    if (col >= dim) continue;
    x[u].load(o, row * dim + col);
    g[u].load(gate, row * ldg + col);
    ss += x[u].squares();
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) s_sum[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int i = 0; i < static_cast<int>(blockDim.x) / 32; ++i) ss += s_sum[i];
  const float r = 1.f / sqrtf(ss / static_cast<float>(dim) + eps);
#pragma unroll
  for (int u = 0; u < kU; ++u) {
    const int col = (threadIdx.x + u * blockDim.x) * 8;
    if (col >= dim) continue;
    x[u].finish(r, g[u], w, w_f32, col, act);
    x[u].store(y, row * dim + col);
  }
}

// x <- silu(x) for the first `cols` elements of every row, in place
template <typename T>
__global__ void __launch_bounds__(256) silu_kernel(T* __restrict__ x, long long ld, int cols, long long total, int vec) {
  const long long step = static_cast<long long>(gridDim.x) * 256;
  for (long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x; i < total; i += step) {
    if (vec) {  // bf16, 8 at a time
      const int per = cols / 8;
      const long long r = i / per;
      uint4* at = reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(x) + r * ld) + (i - r * per);
      uint4 w = *at;
      uint32_t* u = reinterpret_cast<uint32_t*>(&w);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u[e]));
        u[e] = pack_bf16x2(__fdividef(f.x, 1.f + __expf(-f.x)), __fdividef(f.y, 1.f + __expf(-f.y)));
      }
      *at = w;
    } else {
      const long long r = i / cols;
      T* at = x + r * ld + (i - r * cols);
      const float f = to_f(*at);
      store1(at, f / (1.f + expf(-f)));
    }
  }
}

}  // namespace linattn
}  // namespace lvb

// Rows of a piece of lvb_linear_attention's chunked form, and the work items that scratch [items, H, dk, dv] (fp32) is needed for: 0, and a piece of
// at least T rows, when sequences are not to be cut.  longest: rows of the longest sequence (0: not known, or T); only the speed depends on it.
extern "C" int lvb_linear_attention_plan(int T, int longest, int H, int dv, int S, int* piece, int* items) {
  using namespace lvb;
  using namespace lvb::linattn;
  if (T <= 0 || H <= 0 || dv <= 0 || S <= 0) return kErrBadArg;
  if (longest <= 0 || longest > T) longest = T;
  // rounds of the SMs times the chunks that each walks (and one for the start); cut sequences cost two more launches and a pass over what
  // lies before their last pieces, at about half the work per chunk
  const long long slices = static_cast<long long>(H) * ((dv + 63) / 64), sms = num_sms(), seqs = (T + longest - 1) / longest;
  auto rounds = [&](long long pieces) { return (pieces * slices + sms - 1) / sms; };
  long long best = -1;
  int n = 0;
  for (int rows = 256;; rows *= 2) {
    const bool whole = rows >= longest;
    const long long per = whole ? 1 : (longest + rows - 1) / rows, chunks = ((whole ? longest : rows) + 127) / 128;
    const long long cost = 2 * rounds(seqs * per) * (chunks + 1) + (whole ? 0 : rounds(seqs * (per - 1)) * (chunks + 2) + 24);
    if (best < 0 || cost < best) {
      best = cost;
      n = whole ? 0 : rows;
    }
    if (whole) break;
  }
  *piece = n > 0 ? n : (T + 127) / 128 * 128;
  *items = n > 0 ? (T + n - 1) / n + (S < T ? S : T) : 0;
  return kErrOk;
}

// q, k: rows of H * dk, v: rows of H * dv elements (one row stride ld); out [T, H * dv]; fp32 or bf16 (is_f32).  state fp32 [slots, H, dk, dv]: row
// slot_ids[i] belongs to the i-th of num_seqs[0] <= S packed sequences (rows cu_q_lens[i] .. cu_q_lens[i + 1], the last at position kv_lens[i]
// - 1) and is updated in place; a sequence that starts here starts from zeros.  Rows of no sequence come out as zeros.  decay fp32 [H].
// silu: q, k and v pass through silu first (row by row form only).  chunked: sequences of many rows are expected; bf16, dk <= 256, dk, dv and ld
// multiples of 8, q, k, v 16-byte aligned; piece and pieces as lvb_linear_attention_plan says (pieces may be null when its items are 0).
extern "C" int lvb_linear_attention(const void* q, const void* k, const void* v, void* out, const float* decay, float* state, const int* slot_ids,
                                    const int* kv_lens, const int* cu_q_lens, const int* num_seqs, float* pieces, int T, int H, int dk, int dv,
                                    long long ld, int S, int slots, int piece, float key_scale, int silu, int is_f32, int chunked, int* status,
                                    void* stream) {
  using namespace lvb;
  using namespace lvb::linattn;
  if (T <= 0) return kErrOk;
  if (H <= 0 || dk <= 0 || dv <= 0 || S <= 0 || slots <= 0) return kErrBadArg;
  if (H > 65535 || S >= 65535) return kErrTooLarge;
  Params p{q, k, v, out, decay, state, slot_ids, kv_lens, cu_q_lens, num_seqs, pieces, ld, T, H, dk, dv, S, slots, piece, key_scale, silu, status};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (!chunked) return is_f32 ? run_steps<float>(p, s) : run_steps<__nv_bfloat16>(p, s);
  if (is_f32 || silu || ((dk | dv | ld) & 7) || piece <= 0 || piece % kC != 0 ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15))
    return kErrBadArg;
  if (pieces == nullptr && T > piece) return kErrBadArg;
  const int items = (T + piece - 1) / piece + (S < T ? S : T);
  if (dk <= 128) return run_umma(p, items, s);
  if (dk <= 256) return run_chunks<256, 32>(p, items, s);
  return kErrTooLarge;
}

// y [T, dim]: o [T, dim] with every group of dim / groups elements divided by its root mean square, times w [dim] (optional), times the silu (act 0) or the
// sigmoid (act 1) of gate (row stride ldg).  o, gate and y have one type.
extern "C" int lvb_gated_norm(const void* o, const void* gate, long long ldg, const void* w, int w_f32, void* y, int is_f32, int T, int dim, int groups,
                              float eps, int act, void* stream) {
  using namespace lvb;
  using namespace lvb::linattn;
  if (T <= 0) return kErrOk;
  if (dim <= 0 || groups <= 0 || dim % groups != 0 || act < 0 || act > 1) return kErrBadArg;
  const int part = dim / groups;
  const uintptr_t mis = reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(y);
  const int vec = (part & 3) == 0 && (ldg & 3) == 0 && (mis & 15) == 0 ? 4 : 1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (!is_f32 && ((part | ldg) & 7) == 0 && (mis & 15) == 0) {
    const int lanes = part / 8;
    if (lanes <= 32 && (lanes & (lanes - 1)) == 0) {
      const long long units = static_cast<long long>(T) * (dim / 8), cap = static_cast<long long>(num_sms()) * 32;
      const long long blocks = (units + 255) / 256;
      gated_norm_small_kernel<<<static_cast<int>(blocks < cap ? blocks : cap), 256, 0, s>>>(o, gate, ldg, w, w_f32, y, units, dim / 8, lanes, eps, act);
      return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
    }
    if (groups == 1 && dim <= 512 * 32) {
      const int per = dim / 8 <= 512 ? 1 : dim / 8 <= 1024 ? 2 : 4, threads = ((dim / 8 + per - 1) / per + 31) / 32 * 32;
      auto kern = per == 1 ? gated_norm_row_kernel<1> : per == 2 ? gated_norm_row_kernel<2> : gated_norm_row_kernel<4>;
      kern<<<T, threads, 0, s>>>(o, gate, ldg, w, w_f32, y, dim, eps, act);
      return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
    }
  }
  int n, threads;
  if (!rowg::shape_for(dim, vec, T < 2 * num_sms(), n, threads)) return kErrTooLarge;
  auto launch = [&](auto kern, size_t floats) {
    if (floats * 4 > 200 * 1024) return kErrTooLarge;
    if (floats * 4 > 40 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return kErrCuda;
    kern<<<T, threads, floats * 4, s>>>(o, gate, ldg, w, w_f32, y, is_f32, dim, part, eps, act);
    return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
  };
  if (vec == 4) {
    if (n == 1) return launch(gated_norm_kernel<1, 4, 1024>, rowg::Row<1, 4>::scratch_floats(threads, groups));
    if (n == 2) return launch(gated_norm_kernel<2, 4, 512>, rowg::Row<2, 4>::scratch_floats(threads, groups));
    if (n == 4) return launch(gated_norm_kernel<4, 4, 1024>, rowg::Row<4, 4>::scratch_floats(threads, groups));
    return kErrTooLarge;
  }
  if (n == 1) return launch(gated_norm_kernel<1, 1, 1024>, rowg::Row<1, 1>::scratch_floats(threads, groups));
  if (n == 2) return launch(gated_norm_kernel<2, 1, 512>, rowg::Row<2, 1>::scratch_floats(threads, groups));
  if (n == 4) return launch(gated_norm_kernel<4, 1, 1024>, rowg::Row<4, 1>::scratch_floats(threads, groups));
  return launch(gated_norm_kernel<16, 1, 1024>, rowg::Row<16, 1>::scratch_floats(threads, groups));
}

extern "C" int lvb_silu_rows(void* x, long long ld, int rows, int cols, int is_f32, void* stream) {
  using namespace lvb;
  using namespace lvb::linattn;
  if (rows <= 0 || cols <= 0) return kErrOk;
  const int vec = !is_f32 && ((cols | ld) & 7) == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0;
  const long long total = static_cast<long long>(rows) * cols / (vec ? 8 : 1), cap = static_cast<long long>(num_sms()) * 16;
  long long blocks = (total + 255) / 256;
  if (blocks > cap) blocks = cap;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (is_f32) silu_kernel<float><<<static_cast<int>(blocks), 256, 0, s>>>(reinterpret_cast<float*>(x), ld, cols, total, 0);
  else silu_kernel<__nv_bfloat16><<<static_cast<int>(blocks), 256, 0, s>>>(reinterpret_cast<__nv_bfloat16*>(x), ld, cols, total, vec);
  return cudaGetLastError() == cudaSuccess ? kErrOk : kErrCuda;
}
