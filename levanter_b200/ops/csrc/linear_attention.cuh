// What the kernels of linear attention with fixed decays share: their arguments and the cutting of packed sequences into pieces.
#pragma once
#include "common.cuh"

namespace lvb {
namespace linattn {

struct Params {
  const void *q, *k, *v;   // rows of H * dk, H * dk, H * dv elements, row stride ld
  void* out;               // [T, H * dv]
  const float* decay;      // [H]
  float* state;            // [slots, H, dk, dv]
  const int *slot_ids, *kv_lens, *cu_q_lens, *num_seqs;
  float* pieces;           // [work items, H, dk, dv]: what a piece adds to the state, then the state it starts from
  long long ld;
  int T, H, dk, dv, S, slots, piece;  // piece: rows of a piece, a multiple of the chunk
  float key_scale;
  int silu;                // q, k and v pass through silu first (row by row kernel only)
  int* status;
};

// The chunked form for dk <= 128, linear_attention_umma.cu: `items` work items.
int run_umma(const Params& p, int items, cudaStream_t s);
// pieces: what each piece adds -> the state that each piece starts from.
void carry_states(const Params& p, cudaStream_t s);

struct Sequence {
  int r0, r1, slot;
  bool from_state;
};

__device__ __forceinline__ int live_sequences(const Params& p) { return min(p.num_seqs[0], p.S); }

// Rows and slot of sequence i.  False: nothing to do.
__device__ __forceinline__ bool sequence(const Params& p, int i, Sequence& s) {
  s.r0 = max(p.cu_q_lens[i], 0);
  s.r1 = min(p.cu_q_lens[i + 1], p.T);
  s.slot = p.slot_ids[i];
  s.from_state = p.kv_lens[i] > s.r1 - s.r0;
  return s.r1 > s.r0 && s.slot >= 0 && s.slot < p.slots;
}

// Two numbers as two bf16 parts each: hi + lo
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi));
  lo = pack_bf16x2(a - h.x, b - h.y);
}

// Piece of work item w: sequence, number within the sequence and of how many.  A warp's lanes together.  False: there are only `of` items.
__device__ __forceinline__ bool find_piece(const Params& p, int w, int& seq, int& c, int& of) {
  const int lane = threadIdx.x & 31, n_seq = live_sequences(p);
  int before = 0;
  for (int base = 0; base < n_seq; base += 32) {
    const int i = base + lane;
    const int len = i < n_seq ? max(min(p.cu_q_lens[i + 1], p.T) - max(p.cu_q_lens[i], 0), 0) : 0;
    const int n = (len + p.piece - 1) / p.piece;
    int inc = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int u = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += u;
    }
    const bool mine = w >= before + inc - n && w < before + inc;
    const unsigned found = __ballot_sync(0xffffffffu, mine);
    if (found) {
      const int src = __ffs(found) - 1;
      seq = base + src;
      of = __shfl_sync(0xffffffffu, n, src);
      c = w - (before + __shfl_sync(0xffffffffu, inc, src) - of);
      return true;
    }
    before += __shfl_sync(0xffffffffu, inc, 31);
  }
  of = before;
  return false;
}

}  // namespace linattn
}  // namespace lvb
