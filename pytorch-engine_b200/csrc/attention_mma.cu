// Causal grouped-query attention over the paged bfloat16 cache on the tensor cores (mma.sync
// m16n8k16, float32 accumulation), for groups of up to 16 query heads and head sizes 64 and 128 (values of the
// same size), or any key size up to 256 and value size up to 128 that are multiples of 8: those run in tiles of the next
// larger size whose spare columns are zeros (queries: written so; keys and values: TMA fills what lies beyond a row).
// Other shapes and the float32 mode use attention_generic.cu.
//
// Formulas as in attention_generic.cu (pygguf_engine/kv_cache.py:833, 2189-2192 masks; 756 head
// mapping; 836-861 online softmax; 273-282 merge of partial results).  Scores, the softmax state
// (m, l) and the output accumulator are float32; the probabilities are rounded to bfloat16 only as
// the tensor-core operand of the P.V product.
//
// Rows.  For one kv head, a "row" is a (query token, query head of the group) pair: row r is token
// r / group, head r % group.  All rows of a kv head share its keys and values, so the group's heads
// ride along in the M dimension of the MMA instead of re-reading K and V.
//   prefill: a block of 4 warps owns 64 consecutive rows of one (sequence, kv head) and walks the
//            64-key pages of that sequence up to its last row's position; each warp owns 16 rows.
//            K/V pages are double-buffered in shared memory.
//   decode:  one token per sequence, so a kv head has `group` rows (<= 16: one MMA row block).  A block
//            owns one (sequence, kv head, range of `split_keys` keys); its 4 warps each take 16 keys of
//            every 64-key page and are merged at the end; a second kernel merges the ranges.  Which
//            keys a partial result covers depends only on the sequence's own length.
// K/V pages travel from the cache to shared memory by TMA (cp.async.bulk.tensor, one elected thread,
// completion counted on an mbarrier): a page of one kv head is a [64 keys][head_dim] box of a 2-D
// tensor map over the layer's pages, split into 64-feature (128-byte) sub-tiles with the 128-byte
// swizzle, i.e. the 16-byte chunks of a row are XOR-ed with (row & 7).  That makes both the row-wise
// (K) and the transposed (V) ldmatrix reads conflict-free.  Rows of a page beyond the sequence's
// length are not read as zeros: the cache never holds a non-finite value there (the append kernel
// clears the rest of a page when it starts one), and their probabilities are exactly zero.
#include "api.h"
#include "common.cuh"
#include "tma.cuh"

namespace pe {
namespace fa {

constexpr int BN = 64;  // keys per tile = one cache page

struct Args {
  const __nv_bfloat16* q; long long q_ld;
  __nv_bfloat16* out;     long long out_ld;
  int n_heads, n_kv_heads, group;
  float scale_log2;       // softmax scale * log2(e)
  int window;
  const int* seq_qstart; const int* seq_past; const int* seq_slot;
  const int* page_table; int table_stride; int num_pages;
  const __nv_bfloat16* k_pages; const __nv_bfloat16* v_pages;
  int* status;
  float* part_acc; float* part_lse; int split_keys, max_splits, min_range_keys;
  // a sink in the softmax (one added to its denominator) and each head's output turned back by the angle of the
  // query's position (interleaved pairs over the whole head; tables [out_rows, HD/2]); off: 0 and null
  int sink;
  const float* out_cos; const float* out_sin; int out_rows;
  // chunk > 0: a key is visible only inside the query's own block of `chunk` positions (counted from position 0);
  // v_heads: value heads in a page, kv head g reads value head g % v_heads (several key maps over one set of values);
  // out_f32 != 0: `out` is float32 and out_ld counts floats (not with a turned output)
  int chunk, v_heads, out_f32;
  // split_p != 0: a probability enters the P.V product as two bfloat16 terms (its rounding, and the rounding of what
  // that left over), in two products: 16 significant bits of every weight instead of 8
  int split_p;
  // keep_first > 0 (with a window): keys at positions < keep_first stay visible to every later query
  int keep_first;
  // sizes of a key and of a value row; the kernels' tiles are as large or larger
  int hd, vd;
  // each head's output times sigmoid(gate[token, head]) (rows of the step's tokens, gate_ld apart); null: no gate
  const __nv_bfloat16* gate; long long gate_ld;
};

__device__ __forceinline__ float gate_of(const Args& a, int token, int head) {
  return 1.f / (1.f + expf(-__bfloat162float(a.gate[(size_t)token * a.gate_ld + head])));
}

// What rounding (p0, p1) to bfloat16 left over, as a bfloat16 pair.
__device__ __forceinline__ uint32_t pack_bf16_rest(float p0, float p1) {
  const __nv_bfloat162 lead = __floats2bfloat162_rn(p0, p1);
  const __nv_bfloat162 rest = __floats2bfloat162_rn(p0 - __bfloat162float(lead.x), p1 - __bfloat162float(lead.y));
  return *reinterpret_cast<const uint32_t*>(&rest);
}

// First visible key of a query at `qpos` under the window and chunk masks.
__device__ __forceinline__ int first_visible(const Args& a, int qpos) {
  int lo = 0;
  if (a.window > 0) lo = max(lo, qpos - a.window + 1);
  if (a.chunk > 0) lo = max(lo, qpos / a.chunk * a.chunk);
  return lo;
}

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 2^x by the hardware approximation (one instruction, about 2 ulp; exp2(-inf) = 0): the result is
// rounded to bfloat16 or summed into a float32 denominator, so this is within the path's precision.
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

// byte offset of 16-byte chunk `chunk` of row `row` in a [ROWS][HD] bfloat16 tile stored as
// HD/64 sub-tiles of [ROWS][64] with the 128-byte swizzle (the layout TMA writes)
template <int HD, int ROWS = BN> __device__ __forceinline__ uint32_t tile_off(int row, int chunk) {
  return (uint32_t)((chunk >> 3) * (ROWS * 128) + row * 128 + (((chunk & 7) ^ (row & 7)) << 4));
}

// One elected thread starts the copy of one page (64 keys of kv head `kvh`) of K and V into a stage;
// `bar` counts the bytes.
template <int HD, int VD>
__device__ __forceinline__ void issue_page(const Args& a, const CUtensorMap* kmap, const CUtensorMap* vmap, int slot,
                                           int kvh, int k0, char* stage, uint64_t* bar) {
  const int logical = k0 / BN;
  int page = -1;
  if (logical < a.table_stride) page = a.page_table[(size_t)slot * a.table_stride + logical];
  if (page < 0 || page >= a.num_pages) {
    report(a.status, kStatusPageOutOfRange, slot, page, k0);
    page = 0;
  }
  const int y = (page * a.n_kv_heads + kvh) * BN;
  const int yv = (page * a.v_heads + kvh % a.v_heads) * BN;
  tma::mbar_expect_tx(bar, BN * (HD + VD) * 2);
#pragma unroll
  for (int sub = 0; sub < (HD > VD ? HD : VD) / 64; ++sub) {
    if (sub < HD / 64) tma::load_2d(stage + sub * (BN * 128), kmap, sub * 64, y, bar);
    if (sub < VD / 64) tma::load_2d(stage + BN * HD * 2 + sub * (BN * 128), vmap, sub * 64, yv, bar);
  }
}

// A wait ran out: record it, give copies still in flight a last bounded chance to land, and leave.
__device__ __forceinline__ void give_up(const Args& a, uint64_t* bars, int n_bars, int where) {
  if (threadIdx.x == 0) report(a.status, kStatusWaitTimedOut, where, blockIdx.x, blockIdx.z);
  for (int s = 0; s < n_bars; ++s)
    for (int i = 0; i < 1000; ++i)
      if (tma::mbar_try_wait(&bars[s], 0) || tma::mbar_try_wait(&bars[s], 1)) break;
}

__device__ __forceinline__ char* align_1024(char* p) {
  return reinterpret_cast<char*>((reinterpret_cast<uintptr_t>(p) + 1023) & ~static_cast<uintptr_t>(1023));
}

// ---- prefill ---------------------------------------------------------------------------------------
// grid: (row tiles of 64, n_kv_heads, n_seqs); block: 128 threads.
// PAD: rows are a.hd and a.vd features, fewer than the tiles' HD and VD.
template <int HD, int VD, bool SPLIT_P, bool PAD>
__global__ void __launch_bounds__(128, (SPLIT_P || HD > 128) ? 2 : 3) prefill_kernel(Args a, const __grid_constant__ CUtensorMap kmap,
                                                      const __grid_constant__ CUtensorMap vmap) {
  extern __shared__ char smem_raw[];
  __shared__ uint64_t bars[2];
  pdl_wait_block();
  pdl_launch_dependents();
  char* smem = align_1024(smem_raw);
  constexpr int STAGE = BN * (HD + VD) * 2;   // K and V tile
  constexpr int KS = HD / 16;                 // k-steps of Q.K^T
  constexpr int NO = VD / 8;                  // n-tiles of the output
  const int hd = PAD ? a.hd : HD, vd = PAD ? a.vd : VD;
  // Q is staged in the second K/V stage: its fragments are in registers before that stage is first filled (64 rows of
  // HD features fit there: the stage holds that many of K alone)
  char* q_s = smem + STAGE;                   // [64][HD] swizzled
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3;
  const int b = blockIdx.z, kvh = blockIdx.y;
  const int q0 = a.seq_qstart[b], q_len = a.seq_qstart[b + 1] - q0, past = a.seq_past[b];
  const int group = a.group;
  const int n_rows = q_len * group;
  // late rows see the most keys: they go first, so that the longest blocks do not form the tail
  const int row0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * 64;
  if (row0 >= n_rows) return;
  const int slot = a.seq_slot[b];
  const int last_row = min(n_rows, row0 + 64) - 1;
  const int first_pos = past + row0 / group, last_pos = past + last_row / group;
  const int k_begin = first_visible(a, first_pos) / BN * BN;
  const int k_end = last_pos + 1;
  // kept first keys in front of the block's window: their pages come first, then the pages from k_begin on
  const int keep_tiles = a.keep_first > 0 ? (min(a.keep_first, k_begin) + BN - 1) / BN : 0;
  const int n_tiles = keep_tiles + (k_end - k_begin + BN - 1) / BN;
  auto tile_k0 = [&](int it) { return it < keep_tiles ? it * BN : k_begin + (it - keep_tiles) * BN; };

  // first K/V page in flight, then stage Q
  if (tid == 0) {
    tma::mbar_init(&bars[0], 1);
    tma::mbar_init(&bars[1], 1);
    tma::fence_barrier_init();
    issue_page<HD, VD>(a, &kmap, &vmap, slot, kvh, tile_k0(0), smem, &bars[0]);
  }
  constexpr int CPR = HD / 8;
  for (int i = tid; i < 64 * CPR; i += 128) {
    const int r = i / CPR, chunk = i % CPR;
    const int row = row0 + r;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (row < n_rows && (!PAD || chunk * 8 < hd)) {
      const int tok = row / group, head = kvh * group + row % group;
      v = *reinterpret_cast<const uint4*>(a.q + (size_t)(q0 + tok) * a.q_ld + (size_t)head * hd + chunk * 8);
    }
    *reinterpret_cast<uint4*>(q_s + tile_off<HD>(r, chunk)) = v;
  }
  __syncthreads();
  uint32_t qf[KS][4];
#pragma unroll
  for (int ks = 0; ks < KS; ++ks) {
    const int r = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
    ldmatrix_x4(qf[ks], smem_u32(q_s) + tile_off<HD>(r, ks * 2 + (lane >> 4)));
  }
  __syncthreads();  // every warp has its Q fragments: the stage that held Q may now be filled with keys
  // this thread's two rows
  const int r_lo = row0 + warp * 16 + g, r_hi = r_lo + 8;
  const int pos_lo = past + r_lo / group, pos_hi = past + r_hi / group;   // rows beyond n_rows are never stored
  const int warp_last_pos = past + min(n_rows - 1, row0 + warp * 16 + 15) / group;
  const int warp_first_pos = past + min(n_rows - 1, row0 + warp * 16) / group;
  const int warp_first_lo = first_visible(a, warp_first_pos), warp_last_lo = first_visible(a, warp_last_pos);
  const int lo_lo = first_visible(a, pos_lo), lo_hi = first_visible(a, pos_hi);
  float o[NO][4];
#pragma unroll
  for (int n = 0; n < NO; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;

  for (int it = 0; it < n_tiles; ++it) {
    const int k0 = tile_k0(it);
    char* stage = smem + (it & 1) * STAGE;
    // next page into the other stage (everyone left it at the end of the last round)
    if (tid == 0 && it + 1 < n_tiles)
      issue_page<HD, VD>(a, &kmap, &vmap, slot, kvh, tile_k0(it + 1), smem + ((it + 1) & 1) * STAGE, &bars[(it + 1) & 1]);
    if (!tma::mbar_wait(&bars[it & 1], (it >> 1) & 1)) {
      give_up(a, bars, 2, 1);
      return;
    }
    const bool skip = (k0 > warp_last_pos) || (k0 + BN - 1 < warp_first_lo && k0 >= a.keep_first);
    if (!skip) {
      const uint32_t ks_base = smem_u32(stage), vs_base = ks_base + BN * HD * 2;
      float s[8][4];
#pragma unroll
      for (int n = 0; n < 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
#pragma unroll
        for (int np = 0; np < 4; ++np) {  // pairs of 8-key n-tiles
          uint32_t kb[4];
          const int key = np * 16 + (lane & 7) + (lane >> 4) * 8;
          ldmatrix_x4(kb, ks_base + tile_off<HD>(key, ks * 2 + ((lane >> 3) & 1)));
          mma_bf16(s[np * 2], qf[ks], kb[0], kb[1]);
          mma_bf16(s[np * 2 + 1], qf[ks], kb[2], kb[3]);
        }
      }
      // scale, mask, running max
      float mx_lo = -INFINITY, mx_hi = -INFINITY;
      // a page that lies wholly in the past of every row of this warp (and inside every window) needs no mask
      const bool full = (k0 + BN - 1 <= warp_first_pos) && (k0 >= warp_last_lo);
      if (full) {
#pragma unroll
        for (int n = 0; n < 8; ++n) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float v = s[n][e] * a.scale_log2;
            s[n][e] = v;
            if (e < 2) mx_lo = fmaxf(mx_lo, v); else mx_hi = fmaxf(mx_hi, v);
          }
        }
      } else {
#pragma unroll
        for (int n = 0; n < 8; ++n) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int kpos = k0 + n * 8 + 2 * t + (e & 1);
            const int qpos = (e < 2) ? pos_lo : pos_hi;
            const bool vis = kpos <= qpos && (kpos >= ((e < 2) ? lo_lo : lo_hi) || kpos < a.keep_first);
            const float v = vis ? s[n][e] * a.scale_log2 : -INFINITY;
            s[n][e] = v;
            if (e < 2) mx_lo = fmaxf(mx_lo, v); else mx_hi = fmaxf(mx_hi, v);
          }
        }
      }
      mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
      mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
      mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
      mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
      const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);
      const float al_lo = (m_lo == -INFINITY) ? 0.f : fast_exp2(m_lo - mn_lo);
      const float al_hi = (m_hi == -INFINITY) ? 0.f : fast_exp2(m_hi - mn_hi);
      const float base_lo = (mn_lo == -INFINITY) ? 0.f : mn_lo, base_hi = (mn_hi == -INFINITY) ? 0.f : mn_hi;
      float sum_lo = 0.f, sum_hi = 0.f;
      uint32_t pf[4][4];  // P as A operand: 4 k-steps of 16 keys
      uint32_t pr[SPLIT_P ? 4 : 1][4];  // what its rounding left over
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        const float p0 = fast_exp2(s[n][0] - base_lo), p1 = fast_exp2(s[n][1] - base_lo);
        const float p2 = fast_exp2(s[n][2] - base_hi), p3 = fast_exp2(s[n][3] - base_hi);
        sum_lo += p0 + p1;
        sum_hi += p2 + p3;
        pf[n >> 1][(n & 1) * 2] = pack_bf16(p0, p1);
        pf[n >> 1][(n & 1) * 2 + 1] = pack_bf16(p2, p3);
        if (SPLIT_P) {
          pr[n >> 1][(n & 1) * 2] = pack_bf16_rest(p0, p1);
          pr[n >> 1][(n & 1) * 2 + 1] = pack_bf16_rest(p2, p3);
        }
      }
      sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, 1);
      sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, 2);
      sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, 1);
      sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, 2);
      l_lo = l_lo * al_lo + sum_lo;
      l_hi = l_hi * al_hi + sum_hi;
      m_lo = mn_lo;
      m_hi = mn_hi;
#pragma unroll
      for (int n = 0; n < NO; ++n) {
        o[n][0] *= al_lo; o[n][1] *= al_lo; o[n][2] *= al_hi; o[n][3] *= al_hi;
      }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {       // 16 keys per step
#pragma unroll
        for (int np = 0; np < NO / 2; ++np) {  // pairs of 8-feature n-tiles
          uint32_t vb[4];
          const int key = kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
          ldmatrix_x4_trans(vb, vs_base + tile_off<VD>(key, np * 2 + (lane >> 4)));
          mma_bf16(o[np * 2], pf[kk], vb[0], vb[1]);
          mma_bf16(o[np * 2 + 1], pf[kk], vb[2], vb[3]);
          if (SPLIT_P) {
            mma_bf16(o[np * 2], pr[kk], vb[0], vb[1]);
            mma_bf16(o[np * 2 + 1], pr[kk], vb[2], vb[3]);
          }
        }
      }
    }
    __syncthreads();  // the stage may be overwritten in the next round
  }
  if (a.sink) {   // the sink's score is 0: its weight relative to the running maximum (in powers of two)
    l_lo += fast_exp2(-m_lo);
    l_hi += fast_exp2(-m_hi);
  }
  const float inv_lo = 1.f / fmaxf(l_lo, 1e-20f), inv_hi = 1.f / fmaxf(l_hi, 1e-20f);
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int row = half ? r_hi : r_lo;
    if (row >= n_rows) continue;
    const int tok = row / group, head = kvh * group + row % group;
    __nv_bfloat16* dst = a.out + (size_t)(q0 + tok) * a.out_ld + (size_t)head * vd;
    float inv = half ? inv_hi : inv_lo;
    if (a.gate) inv *= gate_of(a, q0 + tok, head);
    if (a.out_cos) {
      // a thread's two adjacent features are one interleaved pair: pair n*4 + t turns back by the position's angle
      const int pos = half ? pos_hi : pos_lo;
      if (pos < 0 || pos >= a.out_rows) {
        report(a.status, kStatusPositionOutOfRange, q0 + tok, pos, a.out_rows);
        continue;
      }
      const float* cs = a.out_cos + (size_t)pos * (VD / 2);
      const float* sn = a.out_sin + (size_t)pos * (VD / 2);
#pragma unroll
      for (int n = 0; n < NO; ++n) {
        const float c = cs[n * 4 + t], sv = sn[n * 4 + t];
        const float x0 = o[n][half * 2] * inv, x1 = o[n][half * 2 + 1] * inv;
        *reinterpret_cast<uint32_t*>(dst + n * 8 + 2 * t) = pack_bf16(x0 * c + x1 * sv, x1 * c - x0 * sv);
      }
      continue;
    }
    if (a.out_f32) {
      float* dstf = reinterpret_cast<float*>(a.out) + (size_t)(q0 + tok) * a.out_ld + (size_t)head * vd;
#pragma unroll
      for (int n = 0; n < NO; ++n)
        if (!PAD || n * 8 < vd) *reinterpret_cast<float2*>(dstf + n * 8 + 2 * t) = make_float2(o[n][half * 2] * inv, o[n][half * 2 + 1] * inv);
      continue;
    }
#pragma unroll
    for (int n = 0; n < NO; ++n) {
      const uint32_t v = pack_bf16(o[n][half * 2] * inv, o[n][half * 2 + 1] * inv);
      if (!PAD || n * 8 < vd) *reinterpret_cast<uint32_t*>(dst + n * 8 + 2 * t) = v;
    }
  }
}

// One warp folds its 16 keys (key0 .. key0+15 of the page that starts at position k0) into the
// running softmax state of the group's rows.  Keys outside [k_first, k_hi) and keys inside [hole_lo, hole_hi) (what lies
// between the kept first keys and the window) are masked.
template <int HD, int VD, bool SPLIT_P>
__device__ __forceinline__ void decode_fold_page(uint32_t ks_base, uint32_t vs_base, int key0, int k0, int k_first,
                                                 int k_hi, int hole_lo, int hole_hi, float scale_log2,
                                                 const uint32_t (&qf)[HD / 16][4],
                                                 float (&o)[VD / 8][4], float& m_lo, float& m_hi, float& l_lo,
                                                 float& l_hi, int lane) {
  constexpr int KS = HD / 16;
  constexpr int NO = VD / 8;
  const int t = lane & 3;
    if (k0 + key0 < k_hi && k0 + key0 + 15 >= k_first && !(k0 + key0 >= hole_lo && k0 + key0 + 15 < hole_hi)) {
  float s[2][4];
  s[0][0] = s[0][1] = s[0][2] = s[0][3] = s[1][0] = s[1][1] = s[1][2] = s[1][3] = 0.f;
#pragma unroll
  for (int ks = 0; ks < KS; ++ks) {
    uint32_t kb[4];
    const int key = key0 + (lane & 7) + (lane >> 4) * 8;
    ldmatrix_x4(kb, ks_base + tile_off<HD>(key, ks * 2 + ((lane >> 3) & 1)));
    mma_bf16(s[0], qf[ks], kb[0], kb[1]);
    mma_bf16(s[1], qf[ks], kb[2], kb[3]);
  }
  float mx_lo = -INFINITY, mx_hi = -INFINITY;
#pragma unroll
  for (int n = 0; n < 2; ++n) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int kpos = k0 + key0 + n * 8 + 2 * t + (e & 1);
      const bool vis = kpos >= k_first && kpos < k_hi && !(kpos >= hole_lo && kpos < hole_hi);
      const float v = vis ? s[n][e] * scale_log2 : -INFINITY;
      s[n][e] = v;
      if (e < 2) mx_lo = fmaxf(mx_lo, v); else mx_hi = fmaxf(mx_hi, v);
    }
  }
  mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
  mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
  mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
  mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
  const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);
  const float al_lo = (m_lo == -INFINITY) ? 0.f : fast_exp2(m_lo - mn_lo);
  const float al_hi = (m_hi == -INFINITY) ? 0.f : fast_exp2(m_hi - mn_hi);
  const float base_lo = (mn_lo == -INFINITY) ? 0.f : mn_lo, base_hi = (mn_hi == -INFINITY) ? 0.f : mn_hi;
  const float p00 = fast_exp2(s[0][0] - base_lo), p01 = fast_exp2(s[0][1] - base_lo);
  const float p02 = fast_exp2(s[0][2] - base_hi), p03 = fast_exp2(s[0][3] - base_hi);
  const float p10 = fast_exp2(s[1][0] - base_lo), p11 = fast_exp2(s[1][1] - base_lo);
  const float p12 = fast_exp2(s[1][2] - base_hi), p13 = fast_exp2(s[1][3] - base_hi);
  float sum_lo = p00 + p01 + p10 + p11, sum_hi = p02 + p03 + p12 + p13;
  sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, 1);
  sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, 2);
  sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, 1);
  sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, 2);
  l_lo = l_lo * al_lo + sum_lo;
  l_hi = l_hi * al_hi + sum_hi;
  m_lo = mn_lo;
  m_hi = mn_hi;
  uint32_t pf[4];
  pf[0] = pack_bf16(p00, p01); pf[1] = pack_bf16(p02, p03); pf[2] = pack_bf16(p10, p11); pf[3] = pack_bf16(p12, p13);
  uint32_t pr[4] = {0u, 0u, 0u, 0u};
  if (SPLIT_P) {
    pr[0] = pack_bf16_rest(p00, p01); pr[1] = pack_bf16_rest(p02, p03);
    pr[2] = pack_bf16_rest(p10, p11); pr[3] = pack_bf16_rest(p12, p13);
  }
#pragma unroll
  for (int n = 0; n < NO; ++n) {
    o[n][0] *= al_lo; o[n][1] *= al_lo; o[n][2] *= al_hi; o[n][3] *= al_hi;
  }
#pragma unroll
  for (int np = 0; np < NO / 2; ++np) {
    uint32_t vb[4];
    const int key = key0 + (lane & 7) + ((lane >> 3) & 1) * 8;
    ldmatrix_x4_trans(vb, vs_base + tile_off<VD>(key, np * 2 + (lane >> 4)));
    mma_bf16(o[np * 2], pf, vb[0], vb[1]);
    mma_bf16(o[np * 2 + 1], pf, vb[2], vb[3]);
    if (SPLIT_P) {
      mma_bf16(o[np * 2], pr, vb[0], vb[1]);
      mma_bf16(o[np * 2 + 1], pr, vb[2], vb[3]);
    }
  }
}
}

// ---- decode ------------------------------------------------------------------------------------------
// Keys per range of a sequence of `len` keys: the fixed split_keys, or (split_keys == 0) the
// sequence's own length shared out evenly over max_splits ranges, in whole pages, but no fewer than
// min_range_keys.  With even shares a grid sized for the longest possible sequence keeps all its
// blocks busy on shorter ones; the floor keeps a short sequence in a grid sized for a much longer
// one from being cut into ranges of a page or two (its spare blocks return at once).
__device__ __forceinline__ int range_keys(const Args& a, int len) {
  if (a.split_keys > 0) return a.split_keys;
  const int per = (len + a.max_splits - 1) / a.max_splits;
  return max(max(BN, a.min_range_keys), (per + BN - 1) / BN * BN);
}

// grid: (max_splits, n_kv_heads, n_seqs); block: 128 threads; STAGES pages in flight.
template <int HD, int VD, int STAGES, bool SPLIT_P, bool PAD>
__global__ void __launch_bounds__(128) decode_split_kernel(Args a, const __grid_constant__ CUtensorMap kmap,
                                                           const __grid_constant__ CUtensorMap vmap) {
  extern __shared__ char smem_raw[];
  __shared__ uint64_t bars[STAGES];
  // The batch description and every page but the sequence's last were written before the kernel that
  // precedes this one started, so they may be read before the dependency wait; the last page (it gets
  // this step's key) and the queries come from that kernel and are read after it.
  char* smem = align_1024(smem_raw);
  constexpr int STAGE = BN * (HD + VD) * 2;
  constexpr int KS = HD / 16;
  constexpr int NO = VD / 8;
  const int hd = PAD ? a.hd : HD, vd = PAD ? a.vd : VD;
  char* q_s = smem + STAGES * STAGE;  // [16][HD] swizzled
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3;
  const int b = blockIdx.z, kvh = blockIdx.y, split = blockIdx.x;
  const int group = a.group;
  const int tq = a.seq_qstart[b];
  const int len = a.seq_past[b] + 1;
  const int per_range = range_keys(a, len);
  const int k_lo = split * per_range, k_hi = min(len, k_lo + per_range);
  if (k_lo >= len) return;
  const int win_lo = first_visible(a, len - 1);
  const int keep = a.keep_first > 0 ? min(a.keep_first, win_lo) : 0;   // kept first keys in front of the window
  if (k_hi <= win_lo && k_lo >= keep) return;
  const int slot = a.seq_slot[b];
  const int k_first = k_lo < keep ? k_lo : max(k_lo, win_lo);          // first visible key of this range
  // the range's pages: those that hold kept keys (from k_lo on, which is a page's start), then those from the window's
  // first key on; a page that holds both is taken once, with the second lot
  const int k_begin = max(k_lo, win_lo) / BN * BN;
  const int win_tiles = k_hi > win_lo ? (k_hi - k_begin + BN - 1) / BN : 0;
  int keep_tiles = k_lo < keep ? (min(keep, k_hi) - k_lo + BN - 1) / BN : 0;
  if (win_tiles > 0 && k_lo + keep_tiles * BN > k_begin) keep_tiles = (k_begin - k_lo) / BN;
  const int n_tiles = keep_tiles + win_tiles;
  auto tile_k0 = [&](int it) { return it < keep_tiles ? k_lo + it * BN : k_begin + (it - keep_tiles) * BN; };
  const int hole_lo = keep, hole_hi = keep > 0 ? win_lo : 0;
  const int last_page_k0 = (len - 1) / BN * BN;
  if (tid == 0) {
#pragma unroll
    for (int s = 0; s < STAGES; ++s) tma::mbar_init(&bars[s], 1);
    tma::fence_barrier_init();
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s)
      if (s < n_tiles && tile_k0(s) != last_page_k0)
        issue_page<HD, VD>(a, &kmap, &vmap, slot, kvh, tile_k0(s), smem + s * STAGE, &bars[s]);
  }
  pdl_wait_block();
  if (tid == 0) {
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s)
      if (s < n_tiles && tile_k0(s) == last_page_k0)
        issue_page<HD, VD>(a, &kmap, &vmap, slot, kvh, tile_k0(s), smem + s * STAGE, &bars[s]);
  }
  constexpr int CPR = HD / 8;
  for (int i = tid; i < 16 * CPR; i += 128) {
    const int r = i / CPR, chunk = i % CPR;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < group && (!PAD || chunk * 8 < hd))
      v = *reinterpret_cast<const uint4*>(a.q + (size_t)tq * a.q_ld + (size_t)(kvh * group + r) * hd + chunk * 8);
    *reinterpret_cast<uint4*>(q_s + tile_off<HD, 16>(r, chunk)) = v;
  }
  __syncthreads();
  uint32_t qf[KS][4];
#pragma unroll
  for (int ks = 0; ks < KS; ++ks) {
    const int r = (lane & 7) + ((lane >> 3) & 1) * 8;
    ldmatrix_x4(qf[ks], smem_u32(q_s) + tile_off<HD, 16>(r, ks * 2 + (lane >> 4)));
  }
  float o[NO][4];
#pragma unroll
  for (int n = 0; n < NO; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;

  for (int it = 0; it < n_tiles; ++it) {
    // keep STAGES-1 pages in flight (the stage refilled here was released by the last round's barrier)
    const int nxt = it + STAGES - 1;
    if (tid == 0 && nxt < n_tiles)
      issue_page<HD, VD>(a, &kmap, &vmap, slot, kvh, tile_k0(nxt), smem + (nxt % STAGES) * STAGE, &bars[nxt % STAGES]);
    if (!tma::mbar_wait(&bars[it % STAGES], (it / STAGES) & 1)) {
      give_up(a, bars, STAGES, 2);
      return;
    }
    const int k0 = tile_k0(it);
    decode_fold_page<HD, VD, SPLIT_P>(smem_u32(smem + (it % STAGES) * STAGE), smem_u32(smem + (it % STAGES) * STAGE) + BN * HD * 2,
                         warp * 16, k0, k_first, k_hi, hole_lo, hole_hi, a.scale_log2, qf, o, m_lo, m_hi, l_lo, l_hi, lane);
    __syncthreads();
  }
  pdl_launch_dependents();
  // merge the four warps (fixed order) through shared memory laid over the stages
  float* ml = reinterpret_cast<float*>(smem);            // [4 warps][16 rows][2]
  float* acc = ml + 4 * 16 * 2;                          // [4 warps][16 rows][VD]
  if (t == 0) {
    ml[(warp * 16 + g) * 2] = m_lo;     ml[(warp * 16 + g) * 2 + 1] = l_lo;
    ml[(warp * 16 + g + 8) * 2] = m_hi; ml[(warp * 16 + g + 8) * 2 + 1] = l_hi;
  }
#pragma unroll
  for (int n = 0; n < NO; ++n) {
    float* r0 = acc + (size_t)(warp * 16 + g) * VD + n * 8 + 2 * t;
    float* r1 = acc + (size_t)(warp * 16 + g + 8) * VD + n * 8 + 2 * t;
    r0[0] = o[n][0]; r0[1] = o[n][1];
    r1[0] = o[n][2]; r1[1] = o[n][3];
  }
  __syncthreads();
  for (int i = tid; i < group * vd; i += 128) {
    const int r = i / vd, c = i - r * vd;
    float mm = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, ml[(w * 16 + r) * 2]);
    float ll = 0.f, aa = 0.f;
    if (mm != -INFINITY) {
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float mw = ml[(w * 16 + r) * 2];
        const float f = (mw == -INFINITY) ? 0.f : fast_exp2(mw - mm);
        ll += ml[(w * 16 + r) * 2 + 1] * f;
        aa += acc[(size_t)(w * 16 + r) * VD + c] * f;
      }
    }
    const size_t pidx = ((size_t)b * a.n_heads + (kvh * group + r)) * a.max_splits + split;
    a.part_acc[pidx * vd + c] = (ll > 0.f) ? aa / ll : 0.f;
    // log-sum-exp in natural units, as the merge kernel expects: (m + log2 l) * ln 2
    if (c == 0) a.part_lse[pidx] = (ll > 0.f) ? (mm + log2f(ll)) * 0.6931471805599453f : -INFINITY;
  }
}

// grid: (n_heads, n_seqs): merge the ranges of one (sequence, head) (pygguf_engine/kv_cache.py:273-282).
// VD: the size of a value row, 0: a.vd.  GATE: outputs may carry a gate (a.gate).
template <int VD, bool GATE>
__global__ void decode_merge_kernel(Args a) {
  pdl_wait_block();
  pdl_launch_dependents();
  const int b = blockIdx.y, h = blockIdx.x;
  const int vd = VD > 0 ? VD : a.vd;
  const int tq = a.seq_qstart[b];
  const int len = a.seq_past[b] + 1;
  const int per_range = range_keys(a, len);
  int n_splits = (len + per_range - 1) / per_range;
  if (n_splits > a.max_splits) {
    // only with a fixed split_keys: the sequence is longer than split_keys * max_splits keys, for which the
    // split grid has no blocks and the scratch no room; say so and merge what was computed
    if (threadIdx.x == 0) report(a.status, kStatusPositionOutOfRange, b, len - 1, per_range * a.max_splits);
    n_splits = a.max_splits;
  }
  const int win_lo = first_visible(a, len - 1);
  const int first = min(win_lo / per_range, n_splits);
  // ranges in front of the window that hold kept first keys were computed too: [0, kept_ranges)
  const int keep = a.keep_first > 0 ? min(a.keep_first, win_lo) : 0;
  const int kept_ranges = min((keep + per_range - 1) / per_range, first);
  const size_t base = ((size_t)b * a.n_heads + h) * a.max_splits;
  __nv_bfloat16* o = a.out + (size_t)tq * a.out_ld + (size_t)h * vd;
  const float gate = GATE && a.gate ? gate_of(a, tq, h) : 1.f;
  // Ranges are taken eight at a time: all their loads are issued before the first is used (this kernel
  // is short and a decode step waits for it once per layer), then they are folded into a running
  // maximum, denominator and sum, in range order.
  constexpr int G = 8;
  for (int c = threadIdx.x; c < vd; c += blockDim.x) {
    // with a sink the fold starts from one more range whose log-sum is 0 and whose output is 0
    float mx = a.sink ? 0.f : -INFINITY, denom = a.sink ? 1.f : 0.f, v = 0.f;
    for (int lot = kept_ranges > 0 ? 0 : 1; lot < 2; ++lot)
    for (int s0 = lot ? first : 0, s_end = lot ? n_splits : kept_ranges; s0 < s_end; s0 += G) {
      float e[G], acc[G];
#pragma unroll
      for (int i = 0; i < G; ++i) {
        const bool live = s0 + i < s_end;
        e[i] = live ? a.part_lse[base + s0 + i] : -INFINITY;
        acc[i] = live ? a.part_acc[(base + s0 + i) * vd + c] : 0.f;
      }
      float m_new = mx;
#pragma unroll
      for (int i = 0; i < G; ++i) m_new = fmaxf(m_new, e[i]);
      if (m_new == -INFINITY) continue;
      const float keep = (mx == -INFINITY) ? 0.f : expf(mx - m_new);
      denom *= keep;
      v *= keep;
#pragma unroll
      for (int i = 0; i < G; ++i) {
        const float w = (e[i] == -INFINITY) ? 0.f : expf(e[i] - m_new);
        denom += w;
        v = fmaf(w, acc[i], v);
      }
      mx = m_new;
    }
    v = v / fmaxf(denom, 1e-20f);
    if (GATE) v *= gate;
    if (a.out_cos) {
      // features c and c ^ 1 (adjacent lanes) are one interleaved pair; every lane of the warp is here (turned outputs: 64 or 128
      // features)
      const float other = __shfl_xor_sync(0xffffffffu, v, 1);
      const int pos = len - 1;
      if (pos < 0 || pos >= a.out_rows) {
        if (c == 0) report(a.status, kStatusPositionOutOfRange, tq, pos, a.out_rows);
        continue;
      }
      const float cs = a.out_cos[(size_t)pos * (vd / 2) + (c >> 1)], sn = a.out_sin[(size_t)pos * (vd / 2) + (c >> 1)];
      v = (c & 1) ? v * cs - other * sn : v * cs + other * sn;
    }
    if (a.out_f32) reinterpret_cast<float*>(a.out)[(size_t)tq * a.out_ld + (size_t)h * vd + c] = v;
    else o[c] = __float2bfloat16_rn(v);
  }
}

template <typename K>
static int opt_in(K kernel, size_t bytes) {
  if (bytes > 227 * 1024) return PE_ERR_UNSUPPORTED_SIZE;
  if (bytes > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (e != cudaSuccess) return (int)e;
  }
  return 0;
}

template <int HD, int VD, bool SPLIT_P, bool PAD>
static int launch(const Args& a, bool decode, int n_seqs, int max_q, cudaStream_t stream) {
  constexpr int STAGE = BN * (HD + VD) * 2;
  CUtensorMap kmap, vmap;
  const uint64_t rows = (uint64_t)a.num_pages * a.n_kv_heads * BN;
  int me = tma::make_map_2d_bf16(&kmap, a.k_pages, a.hd, rows, a.hd, 64, BN);
  if (me == 0) me = tma::make_map_2d_bf16(&vmap, a.v_pages, a.vd, (uint64_t)a.num_pages * a.v_heads * BN, a.vd, 64, BN);
  if (me != 0) return me < 0 ? me : PE_ERR_BAD_ARGUMENT;
  if (!decode) {
    const size_t smem = 1024 + 2 * STAGE;
    auto k = prefill_kernel<HD, VD, SPLIT_P, PAD>;
    int e = opt_in(k, smem);
    if (e) return e;
    const long long tiles = ((long long)max_q * a.group + 63) / 64;
    dim3 grid((unsigned)tiles, a.n_kv_heads, n_seqs);
    if (grid.y > 65535 || grid.z > 65535) return PE_ERR_UNSUPPORTED_SIZE;
    pe::launch(k, grid, 128, smem, stream, a, kmap, vmap);
    PE_LAUNCH_CHECK();
    return PE_OK;
  }
  dim3 grid(a.max_splits, a.n_kv_heads, n_seqs);
  if (grid.y > 65535 || grid.z > 65535) return PE_ERR_UNSUPPORTED_SIZE;
  auto go = [&](auto kern, int STAGES) -> int {
    size_t smem = STAGES * STAGE + 16 * HD * 2;
    const size_t merge = (4 * 16 * 2 + 4 * 16 * VD) * sizeof(float);
    if (merge > smem) smem = merge;
    smem += 1024;
    int e = opt_in(kern, smem);
    if (e) return e;
    pe::launch(kern, grid, 128, smem, stream, a, kmap, vmap);
    return 0;
  };
  // three stages: two blocks per SM, two pages in flight per block (measured best of 2, 3, 4)
  const int e = go(decode_split_kernel<HD, VD, 3, SPLIT_P, PAD>, 3);
  if (e) return e;
  PE_LAUNCH_CHECK();
  // The merge starts when the split kernel has completed, not while it drains: with the early start a
  // decode step of the 8B shape took 4.32 instead of 4.03 ms at batch 8 and context 4,096 (3.59 / 3.49 ms
  // at 1,024, 4.92 / 4.74 at 8,192, 3.95 / 3.56 for 16 layers of the 32B shape), and never less, at batch
  // 1 to 64.  Why its waiting blocks cost that much is not known; switching the early start off for any
  // other kernel of the step gained nothing or lost.
  dim3 mgrid(a.n_heads, n_seqs);
  pe::launch_after(a.gate ? decode_merge_kernel<0, true> : decode_merge_kernel<PAD ? 0 : VD, false>, mgrid, a.vd > 64 ? 128 : 64, 0, stream, a);
  PE_LAUNCH_CHECK();
  return PE_OK;
}

}  // namespace fa
}  // namespace pe

// The tile sizes that rows of these sizes run in.
static int tile_of(int dim) { return (dim + 63) / 64 * 64; }

// Decode blocks that one SM holds at a time (shared memory bound): the caller sizes the number of
// ranges per sequence so that one wave of blocks covers the batch.
extern "C" int pe_attention_mma_decode_blocks_per_sm(int head_dim, int v_dim) {
  const size_t hd = tile_of(head_dim), vd = tile_of(v_dim);
  const size_t stage = (size_t)pe::fa::BN * (hd + vd) * 2;
  const size_t smem = 3 * stage + 16 * hd * 2 + 1024 + 1024;   // + the block's static and reserved part
  const int n = (int)((227 * 1024) / smem);
  return n < 1 ? 1 : n;
}

// 1 if this file's kernels take the shape (bfloat16 only), else 0: the caller then uses the generic path.
extern "C" int pe_attention_mma_supported(int head_dim, int n_heads, int n_kv_heads) {
  if (head_dim != 64 && head_dim != 128) return 0;
  if (n_kv_heads <= 0 || n_heads % n_kv_heads) return 0;
  if (n_heads / n_kv_heads > 16) return 0;
  return 1;
}

// The same for keys and values of sizes of their own, which run in padded tiles unless they are both 64 or both 128.
extern "C" int pe_attention_mma_dims_supported(int head_dim, int v_dim, int n_heads, int n_kv_heads) {
  if (head_dim < 8 || head_dim > 256 || head_dim % 8 || v_dim < 8 || v_dim > 128 || v_dim % 8) return 0;
  if (n_kv_heads <= 0 || n_heads % n_kv_heads) return 0;
  return n_heads / n_kv_heads <= 16 ? 1 : 0;
}

extern "C" int pe_attention_mma(int decode, const void* q, long long q_ld, void* out, long long out_ld, int n_seqs,
                                int max_q, int n_heads, int n_kv_heads, int head_dim, float scale, int window,
                                const int* seq_qstart, const int* seq_past, const int* seq_slot, const int* page_table,
                                int table_stride, int num_pages, const void* k_pages, const void* v_pages,
                                float* scratch, int split_keys, int max_splits, int min_range_keys, int* status,
                                cudaStream_t stream) {
  return pe_attention_mma_ex(decode, q, q_ld, out, out_ld, n_seqs, max_q, n_heads, n_kv_heads, head_dim, scale, window, 0,
                             nullptr, nullptr, 0, seq_qstart, seq_past, seq_slot, page_table, table_stride, num_pages,
                             k_pages, v_pages, scratch, split_keys, max_splits, min_range_keys, status, stream);
}

// The same with a sink in the softmax and, with tables, each head's output turned back by the query's position
// (interleaved pairs over the whole head; out_cos, out_sin: float32 [out_rows, head_dim / 2]).
extern "C" int pe_attention_mma_ex(int decode, const void* q, long long q_ld, void* out, long long out_ld, int n_seqs,
                                   int max_q, int n_heads, int n_kv_heads, int head_dim, float scale, int window, int sink,
                                   const float* out_cos, const float* out_sin, int out_rows, const int* seq_qstart,
                                   const int* seq_past, const int* seq_slot, const int* page_table, int table_stride,
                                   int num_pages, const void* k_pages, const void* v_pages, float* scratch,
                                   int split_keys, int max_splits, int min_range_keys, int* status, cudaStream_t stream) {
  return pe_attention_mma_masked(decode, q, q_ld, out, out_ld, n_seqs, max_q, n_heads, n_kv_heads, head_dim, scale, window,
                                 0, 0, n_kv_heads, 0, 0, sink, out_cos, out_sin, out_rows, seq_qstart, seq_past, seq_slot,
                                 page_table, table_stride, num_pages, k_pages, v_pages, scratch, split_keys, max_splits,
                                 min_range_keys, status, stream);
}

// The same with a chunk mask (`chunk` > 0: keys inside the query's own block of that many positions), kept first keys
// (`keep_first` > 0 with a window: positions below it stay visible however far back they lie), `v_heads` value
// heads a page (kv head g reads value head g % v_heads), optionally a float32 output (`out_f32`: out_ld counts floats)
// and optionally (`split_p`) every probability as two bfloat16 terms in the P.V product.
extern "C" int pe_attention_mma_masked(int decode, const void* q, long long q_ld, void* out, long long out_ld, int n_seqs,
                                       int max_q, int n_heads, int n_kv_heads, int head_dim, float scale, int window,
                                       int chunk, int keep_first, int v_heads, int out_f32, int split_p, int sink, const float* out_cos,
                                       const float* out_sin, int out_rows, const int* seq_qstart, const int* seq_past,
                                       const int* seq_slot, const int* page_table, int table_stride, int num_pages,
                                       const void* k_pages, const void* v_pages, float* scratch, int split_keys,
                                       int max_splits, int min_range_keys, int* status, cudaStream_t stream) {
  return pe_attention_mma_gated(decode, q, q_ld, out, out_ld, n_seqs, max_q, n_heads, n_kv_heads, head_dim, head_dim, scale, window,
                                chunk, keep_first, v_heads, out_f32, split_p, sink, out_cos, out_sin, out_rows, nullptr, 0,
                                seq_qstart, seq_past, seq_slot, page_table, table_stride, num_pages, k_pages, v_pages, scratch,
                                split_keys, max_splits, min_range_keys, status, stream);
}

// The same with values of a size of their own (`v_dim`; the scratch of a decode step then holds v_dim floats per partial
// row) and, with `gate` (bfloat16, row of token t at gate + t * gate_ld), each head's output times sigmoid(gate[t, head]).
extern "C" int pe_attention_mma_gated(int decode, const void* q, long long q_ld, void* out, long long out_ld, int n_seqs,
                                      int max_q, int n_heads, int n_kv_heads, int head_dim, int v_dim, float scale, int window,
                                      int chunk, int keep_first, int v_heads, int out_f32, int split_p, int sink,
                                      const float* out_cos, const float* out_sin, int out_rows, const void* gate,
                                      long long gate_ld, const int* seq_qstart, const int* seq_past, const int* seq_slot,
                                      const int* page_table, int table_stride, int num_pages, const void* k_pages,
                                      const void* v_pages, float* scratch, int split_keys, int max_splits, int min_range_keys,
                                      int* status, cudaStream_t stream) {
  if (n_seqs <= 0) return PE_OK;
  const bool exact = head_dim == v_dim && (head_dim == 64 || head_dim == 128);
  if (!exact && (split_p || out_cos)) return PE_ERR_UNSUPPORTED_SIZE;
  if ((out_cos == nullptr) != (out_sin == nullptr)) return PE_ERR_BAD_ARGUMENT;
  if (chunk < 0 || v_heads <= 0 || (out_f32 && out_cos)) return PE_ERR_BAD_ARGUMENT;
  if (keep_first < 0 || (keep_first > 0 && chunk > 0)) return PE_ERR_BAD_ARGUMENT;
  if (!pe_attention_mma_dims_supported(head_dim, v_dim, n_heads, n_kv_heads)) return PE_ERR_UNSUPPORTED_SIZE;
  // 16-byte vector loads of q rows; 4-byte (bfloat16 pairs) or 8-byte (float pairs) stores of output rows
  const int out_bytes = out_f32 ? 4 : 2;
  if ((q_ld * 2) % 16 || ((uintptr_t)q % 16) || (out_ld * out_bytes) % (2 * out_bytes) || ((uintptr_t)out % (2 * out_bytes)))
    return PE_ERR_BAD_ARGUMENT;
  if (((uintptr_t)k_pages % 16) || ((uintptr_t)v_pages % 16)) return PE_ERR_BAD_ARGUMENT;
  pe::fa::Args a;
  a.q = (const __nv_bfloat16*)q; a.q_ld = q_ld; a.out = (__nv_bfloat16*)out; a.out_ld = out_ld;
  a.n_heads = n_heads; a.n_kv_heads = n_kv_heads; a.group = n_heads / n_kv_heads;
  a.scale_log2 = scale * 1.4426950408889634f; a.window = window;
  a.seq_qstart = seq_qstart; a.seq_past = seq_past; a.seq_slot = seq_slot;
  a.page_table = page_table; a.table_stride = table_stride; a.num_pages = num_pages;
  a.k_pages = (const __nv_bfloat16*)k_pages; a.v_pages = (const __nv_bfloat16*)v_pages; a.status = status;
  a.part_acc = nullptr; a.part_lse = nullptr; a.split_keys = 0; a.max_splits = 0; a.min_range_keys = 0;
  a.sink = sink; a.out_cos = out_cos; a.out_sin = out_sin; a.out_rows = out_rows;
  a.chunk = chunk; a.v_heads = v_heads; a.out_f32 = out_f32; a.split_p = split_p;
  a.keep_first = window > 0 ? keep_first : 0;
  a.hd = head_dim; a.vd = v_dim; a.gate = (const __nv_bfloat16*)gate; a.gate_ld = gate_ld;
  if (decode) {
    if (!scratch || split_keys < 0 || split_keys % pe::fa::BN || max_splits <= 0) return PE_ERR_BAD_ARGUMENT;
    if (min_range_keys < 0 || min_range_keys % pe::fa::BN) return PE_ERR_BAD_ARGUMENT;
    a.split_keys = split_keys; a.max_splits = max_splits; a.min_range_keys = min_range_keys;
    a.part_acc = scratch;
    a.part_lse = scratch + (size_t)n_seqs * n_heads * max_splits * v_dim;
  }
  using pe::fa::launch;
  const bool dec = decode != 0;
  if (exact) {
    if (split_p) {
      if (head_dim == 64) return launch<64, 64, true, false>(a, dec, n_seqs, max_q, stream);
      return launch<128, 128, true, false>(a, dec, n_seqs, max_q, stream);
    }
    if (head_dim == 64) return launch<64, 64, false, false>(a, dec, n_seqs, max_q, stream);
    return launch<128, 128, false, false>(a, dec, n_seqs, max_q, stream);
  }
  const bool wide = v_dim > 64;
  switch (tile_of(head_dim)) {
    case 64: return wide ? launch<64, 128, false, true>(a, dec, n_seqs, max_q, stream) : launch<64, 64, false, true>(a, dec, n_seqs, max_q, stream);
    case 128: return wide ? launch<128, 128, false, true>(a, dec, n_seqs, max_q, stream) : launch<128, 64, false, true>(a, dec, n_seqs, max_q, stream);
    case 192: return wide ? launch<192, 128, false, true>(a, dec, n_seqs, max_q, stream) : launch<192, 64, false, true>(a, dec, n_seqs, max_q, stream);
    default: return wide ? launch<256, 128, false, true>(a, dec, n_seqs, max_q, stream) : launch<256, 64, false, true>(a, dec, n_seqs, max_q, stream);
  }
}
