// Per-head q/k RMSNorm, rotary position encoding and the append of k, v to the paged cache, in one
// pass over the fused q|k|v projection; and the small kernel that expands the batch description
// into per-token sequence index and position.
//
// Reference formulas: q/k-norm over head_dim before RoPE, not on v (pygguf_engine/model.py:471-474);
// split-half rotation of the first rotary_dim features with position = cached length + row
// (pygguf_engine/model.py:232-241, 211-214); append at [P, P+S) (pygguf_engine/model.py:482-483);
// positions read from device memory (pygguf_engine/kv_cache.py:1847-1852).
#include "api.h"
#include "common.cuh"

namespace pe {

// token_seq[t] = index of the batch entry that token t belongs to; token_pos[t] = its position.
__global__ void batch_expand_kernel(const int* seq_qstart, const int* seq_past,
                                    int n_seqs, int* __restrict__ token_seq, int* __restrict__ token_pos) {
  pdl_wait_block();
  pdl_launch_dependents();
  const int b = blockIdx.x;
  if (b >= n_seqs) return;
  const int q0 = seq_qstart[b], q1 = seq_qstart[b + 1], past = seq_past[b];
  for (int t = q0 + threadIdx.x; t < q1; t += blockDim.x) {
    token_seq[t] = b;
    token_pos[t] = past + (t - q0);
  }
}

struct RopeAppendArgs {
  void* qkv;            // [n_tokens, ld]; q heads, then k heads, then v heads; q and k are rewritten in place
  long long ld;
  int n_tokens, n_heads, n_kv_heads, head_dim;
  const float* q_norm_w;  // [head_dim] or null
  const float* k_norm_w;  // [head_dim] or null
  float eps;
  const float* cos_table;  // [table_rows, rotary_dim/2] or null
  const float* sin_table;
  int rotary_dim, table_rows;
  const int* token_seq;
  const int* token_pos;
  const int* seq_slot;
  const int* seq_qstart;   // [n_seqs + 1]
  const int* page_table;   // [slots, table_stride]
  int table_stride, num_pages;
  void* k_pages;           // [num_pages, n_kv_heads, 64, head_dim]
  void* v_pages;
  int write_cache;
  int* status;
};

template <typename T> __device__ __forceinline__ float2 load2(const T* p);
template <> __device__ __forceinline__ float2 load2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> __device__ __forceinline__ float2 load2<__nv_bfloat16>(const __nv_bfloat16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
template <typename T> __device__ __forceinline__ void store2(T* p, float2 v);
template <> __device__ __forceinline__ void store2<float>(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
template <> __device__ __forceinline__ void store2<__nv_bfloat16>(__nv_bfloat16* p, float2 v) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y);
}

// PAIRS: every access covers two adjacent features (head size and half the rotary size even, rows
// aligned to two elements); otherwise one feature at a time.
template <typename T, bool PAIRS>
__global__ void qk_norm_rope_append_kernel(RopeAppendArgs a) {
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y * (blockDim.x >> 5) + warp;
  const int total_heads = a.n_heads + 2 * a.n_kv_heads;
  const bool valid = t < a.n_tokens && head < total_heads;
  const int d = a.head_dim;
  const bool is_q = head < a.n_heads;
  const bool is_k = !is_q && head < a.n_heads + a.n_kv_heads;
  const int kv_head = is_q ? -1 : (is_k ? head - a.n_heads : head - a.n_heads - a.n_kv_heads);
  // Before the wait: what does not come from the kernel before this one.  The step's batch description
  // and the page table were complete before that kernel started, the angle tables and norm weights never
  // change; only the q|k|v rows have to be waited for.  In a decode step this kernel's latency is on the
  // critical path, and the chain token -> sequence -> slot -> page is three trips to memory.
  const bool to_cache = valid && !is_q && a.write_cache;
  int pos = 0, seq = 0, slot = 0, q_begin = 0, q_end = 0, page = -1;
  if (valid) pos = a.token_pos[t];
  if (to_cache) {
    seq = a.token_seq[t];
    slot = a.seq_slot[seq];
    q_begin = a.seq_qstart[seq];
    q_end = a.seq_qstart[seq + 1];
    if (pos >= 0 && pos / kPageTokens < a.table_stride)
      page = a.page_table[(size_t)slot * a.table_stride + pos / kPageTokens];
  }
  const float* w = is_q ? a.q_norm_w : a.k_norm_w;
  const int rot = a.cos_table ? a.rotary_dim : 0;
  const int half = rot / 2;
  const bool rotates = valid && (is_q || is_k);
  const bool pos_in_table = pos >= 0 && pos < a.table_rows;
  const float* cs = (rot > 0 && pos_in_table) ? a.cos_table + (size_t)pos * half : nullptr;
  const float* sn = (rot > 0 && pos_in_table) ? a.sin_table + (size_t)pos * half : nullptr;
  // the first pair of each lane (PAIRS): angles and weights are on their way before the wait
  float2 c_first = make_float2(1.f, 1.f), s_first = make_float2(0.f, 0.f);
  float2 w1_first = make_float2(1.f, 1.f), w2_first = make_float2(1.f, 1.f);
  if (PAIRS && rotates && lane * 2 < half) {
    if (cs) {
      c_first = *reinterpret_cast<const float2*>(cs + lane * 2);
      s_first = *reinterpret_cast<const float2*>(sn + lane * 2);
    }
    if (w) {
      w1_first = *reinterpret_cast<const float2*>(w + lane * 2);
      w2_first = *reinterpret_cast<const float2*>(w + lane * 2 + half);
    }
  }
  pdl_wait_block();
  pdl_launch_dependents();
  if (!valid) return;
  T* row = (T*)a.qkv + (size_t)t * a.ld + (size_t)head * d;

  // where this token's k/v row lies in the paged cache
  T* cache_row = nullptr;
  if (to_cache) {
    if (pos < 0 || pos / kPageTokens >= a.table_stride) {
      if (lane == 0) report(a.status, kStatusPositionOutOfRange, t, pos, a.table_stride * kPageTokens);
    } else if (page < 0 || page >= a.num_pages) {
      if (lane == 0) report(a.status, kStatusPageOutOfRange, t, page, a.num_pages);
    } else {
      T* base = (T*)(is_k ? a.k_pages : a.v_pages);
      const int off = pos % kPageTokens;
      cache_row = base + (((size_t)page * a.n_kv_heads + kv_head) * kPageTokens + off) * d;
      // Rows of a page beyond the sequence's last key must hold finite values (readers multiply them
      // by a probability of zero): the sequence's last token of this step clears the rest of its page
      // when it starts the page or ends a multi-token step; later single tokens find it cleared.
      if (t + 1 == q_end && off + 1 < kPageTokens && (off == 0 || q_end - q_begin > 1)) {
        T* rest = cache_row + d;
        const size_t n = (size_t)(kPageTokens - 1 - off) * d;
        if ((d * sizeof(T)) % 16 == 0) {
          uint4* r4 = reinterpret_cast<uint4*>(rest);
          const size_t n4 = n * sizeof(T) / 16;
          for (size_t i = lane; i < n4; i += 32) r4[i] = make_uint4(0, 0, 0, 0);
        } else {
          for (size_t i = lane; i < n; i += 32) rest[i] = from_f32<T>(0.f);
        }
      }
    }
  }

  if (!is_q && !is_k) {  // v: copy only
    if (cache_row) {
      if (PAIRS) {
        for (int c = lane * 2; c < d; c += 64) store2<T>(cache_row + c, load2<T>(row + c));
      } else {
        for (int c = lane; c < d; c += 32) cache_row[c] = row[c];
      }
    }
    return;
  }

  float inv = 1.f;
  if (w) {
    float ss = 0.f;
    if (PAIRS) {
      for (int c = lane * 2; c < d; c += 64) {
        const float2 x = load2<T>(row + c);
        ss += x.x * x.x + x.y * x.y;
      }
    } else {
      for (int c = lane; c < d; c += 32) {
        const float x = to_f32<T>(row[c]);
        ss += x * x;
      }
    }
    ss = warp_sum(ss);
    inv = rsqrtf(ss / (float)d + a.eps);
  }
  // Norm and rotation are one float32 computation: nothing is rounded between them (the reference
  // rounds to its 16-bit type in between only because they are separate ops there).
  auto normed = [&](int c) -> float {
    float x = to_f32<T>(row[c]);
    if (w) x = x * inv * w[c];
    return x;
  };
  if (rot > 0 && !pos_in_table) {
    if (lane == 0) report(a.status, kStatusPositionOutOfRange, t, pos, a.table_rows);
    return;
  }
  if (PAIRS) {
    for (int j = lane * 2; j < half; j += 64) {
      const bool first = j == lane * 2;
      float2 x1 = load2<T>(row + j), x2 = load2<T>(row + j + half);
      if (w) {
        const float2 w1 = first ? w1_first : *reinterpret_cast<const float2*>(w + j);
        const float2 w2 = first ? w2_first : *reinterpret_cast<const float2*>(w + j + half);
        x1.x *= inv * w1.x; x1.y *= inv * w1.y; x2.x *= inv * w2.x; x2.y *= inv * w2.y;
      }
      const float2 c = first ? c_first : *reinterpret_cast<const float2*>(cs + j);
      const float2 sv = first ? s_first : *reinterpret_cast<const float2*>(sn + j);
      const float2 o1 = make_float2(x1.x * c.x - x2.x * sv.x, x1.y * c.y - x2.y * sv.y);
      const float2 o2 = make_float2(x2.x * c.x + x1.x * sv.x, x2.y * c.y + x1.y * sv.y);
      store2<T>(row + j, o1);
      store2<T>(row + j + half, o2);
      if (cache_row) {
        store2<T>(cache_row + j, o1);
        store2<T>(cache_row + j + half, o2);
      }
    }
    for (int c = rot + lane * 2; c < d; c += 64) {
      float2 x = load2<T>(row + c);
      if (w) {
        const float2 wv = *reinterpret_cast<const float2*>(w + c);
        x.x *= inv * wv.x; x.y *= inv * wv.y;
      }
      store2<T>(row + c, x);
      if (cache_row) store2<T>(cache_row + c, x);
    }
    return;
  }
  // rotated pairs (j, j + half): both are read before either is written
  for (int j = lane; j < half; j += 32) {
    const float x1 = normed(j), x2 = normed(j + half);
    const float c = cs[j], s = sn[j];
    const T o1 = from_f32<T>(x1 * c - x2 * s);
    const T o2 = from_f32<T>(x2 * c + x1 * s);
    row[j] = o1;
    row[j + half] = o2;
    if (cache_row) {
      cache_row[j] = o1;
      cache_row[j + half] = o2;
    }
  }
  // features beyond rotary_dim pass through (normalised only)
  for (int c = rot + lane; c < d; c += 32) {
    const T o = from_f32<T>(normed(c));
    row[c] = o;
    if (cache_row) cache_row[c] = o;
  }
}

// The same for bfloat16 rows with 16-byte accesses: head sizes that are multiples of 16 up to 256,
// the whole head rotated, everything 16-byte aligned.  A head takes head_dim / 8 lanes, so a warp
// holds several heads; the lane that holds features [8i, 8i + 8) of the first half trades its
// normalised values with the lane that holds the matching features of the second half.  A block
// takes TPB tokens and asks for all their rows and positions before it uses the first: a thread
// with one 16-byte load in flight at a time reached 2.3 TB/s on a 2,048-token step (54 MB moved in
// 23.6 us), which is the latency of one load after the other, not bandwidth.
template <int TPB>
__global__ void __launch_bounds__(256, 4) qk_norm_rope_append_vec8_kernel(RopeAppendArgs a, int lanes_per_head) {
  pdl_wait_block();
  pdl_launch_dependents();
  typedef __nv_bfloat16 T;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int lph = lanes_per_head, heads_per_warp = 32 / lph;
  const int sub = lane / lph, li = lane - sub * lph;
  const int total_heads = a.n_heads + 2 * a.n_kv_heads;
  const int head = (blockIdx.y * (blockDim.x >> 5) + warp) * heads_per_warp + sub;
  const bool active = sub < heads_per_warp && head < total_heads;
  const int d = a.head_dim;
  const bool is_q = head < a.n_heads;
  const bool is_k = !is_q && head < a.n_heads + a.n_kv_heads;
  const bool is_v = !is_q && !is_k;
  const int kv_head = is_k ? head - a.n_heads : head - a.n_heads - a.n_kv_heads;
  const int half_l = lph >> 1;
  const bool second = li >= half_l;
  const int j = 8 * (second ? li - half_l : li);  // this lane's place in a row of the angle tables
  const int partner = lane + (second ? -half_l : half_l);
  const bool pow2 = (lph & (lph - 1)) == 0;
  const bool rotate = a.cos_table != nullptr && a.rotary_dim > 0;
  const float* w = is_q ? a.q_norm_w : a.k_norm_w;
  float wv[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) wv[e] = 1.f;
  if (active && !is_v && w) {
    const float4 w0 = *reinterpret_cast<const float4*>(w + 8 * li), w1 = *reinterpret_cast<const float4*>(w + 8 * li + 4);
    wv[0] = w0.x; wv[1] = w0.y; wv[2] = w0.z; wv[3] = w0.w; wv[4] = w1.x; wv[5] = w1.y; wv[6] = w1.z; wv[7] = w1.w;
  }
  // every token's row and position first: independent loads, all in flight together
  uint4 raws[TPB];
  int poss[TPB];
#pragma unroll
  for (int i = 0; i < TPB; ++i) {
    const int t = blockIdx.x * TPB + i;
    raws[i] = make_uint4(0, 0, 0, 0);
    poss[i] = -1;
    if (t < a.n_tokens) {
      if (active) raws[i] = *reinterpret_cast<const uint4*>((const T*)a.qkv + (size_t)t * a.ld + (size_t)head * d + 8 * li);
      poss[i] = a.token_pos[t];
    }
  }
#pragma unroll
  for (int i = 0; i < TPB; ++i) {
    const int t = blockIdx.x * TPB + i;
    if (t >= a.n_tokens) break;
    T* row = (T*)a.qkv + (size_t)t * a.ld + (size_t)head * d + 8 * li;
    const uint4 raw = raws[i];
    const int pos = poss[i];
    T* cache_row = nullptr;
    if (active && !is_q && a.write_cache) {
      const int b = a.token_seq[t];
      const int slot = a.seq_slot[b];
      const int logical = pos / kPageTokens;
      if (pos < 0 || logical >= a.table_stride) {
        if (li == 0) report(a.status, kStatusPositionOutOfRange, t, pos, a.table_stride * kPageTokens);
      } else {
        const int page = a.page_table[(size_t)slot * a.table_stride + logical];
        if (page < 0 || page >= a.num_pages) {
          if (li == 0) report(a.status, kStatusPageOutOfRange, t, page, a.num_pages);
        } else {
          T* base = (T*)(is_k ? a.k_pages : a.v_pages);
          const int off = pos % kPageTokens;
          T* head_row = base + (((size_t)page * a.n_kv_heads + kv_head) * kPageTokens + off) * d;
          cache_row = head_row + 8 * li;
          // clear the rest of the page (see the kernel above for when and why)
          const int q_end = a.seq_qstart[b + 1];
          if (t + 1 == q_end && off + 1 < kPageTokens && (off == 0 || q_end - a.seq_qstart[b] > 1)) {
            uint4* r4 = reinterpret_cast<uint4*>(head_row + d);
            const size_t n4 = (size_t)(kPageTokens - 1 - off) * d / 8;
            for (size_t x = li; x < n4; x += lph) r4[x] = make_uint4(0, 0, 0, 0);
          }
        }
      }
    }
    float x[8];
    {
      const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(h2[e]);
        x[2 * e] = f.x;
        x[2 * e + 1] = f.y;
      }
    }
    {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
      if (pow2) {
        for (int o = lph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      } else {
        float total = 0.f;
        for (int l = 0; l < lph; ++l) total += __shfl_sync(0xffffffffu, ss, (sub * lph + l) & 31);
        ss = total;
      }
      if (!is_v && w != nullptr) {
        const float inv = rsqrtf(ss / (float)d + a.eps);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = x[e] * inv * wv[e];
      }
    }
    float other[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) other[e] = __shfl_sync(0xffffffffu, x[e], partner & 31);
    if (active && !is_v && rotate) {
      if (pos < 0 || pos >= a.table_rows) {
        if (li == 0) report(a.status, kStatusPositionOutOfRange, t, pos, a.table_rows);
        continue;
      }
      const float* cs = a.cos_table + (size_t)pos * (d / 2) + j;     // the tables stay in L2
      const float* sn = a.sin_table + (size_t)pos * (d / 2) + j;
      const float4 c0 = *reinterpret_cast<const float4*>(cs), c1 = *reinterpret_cast<const float4*>(cs + 4);
      const float4 s0 = *reinterpret_cast<const float4*>(sn), s1 = *reinterpret_cast<const float4*>(sn + 4);
      const float cv[8] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w};
      const float sv[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] = second ? x[e] * cv[e] + other[e] * sv[e] : x[e] * cv[e] - other[e] * sv[e];
    }
    if (!active) continue;
    uint4 out = raw;
    if (!is_v) {
      __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
      for (int e = 0; e < 4; ++e) o2[e] = __floats2bfloat162_rn(x[2 * e], x[2 * e + 1]);
      *reinterpret_cast<uint4*>(row) = out;
    }
    if (cache_row) *reinterpret_cast<uint4*>(cache_row) = out;
  }
}

// ---- the general form -------------------------------------------------------------------------------------------
// Queries and keys: optional RMS norm with a weight, then rotation of the first `rotary_dim` features in either
// layout of pairs (split-half: j with j + rotary_dim/2; interleaved: 2j with 2j + 1), angle tables by position (a
// table may carry a factor on cos and sin).  Values, of a size of their own: optionally divided by their root mean
// square (no weight), optionally rotated by their position over `v_rotary_dim` features with tables of their own;
// they go to the cache so.  One warp per (token, head), float32 arithmetic, any sizes.
struct QkvRotateArgs {
  void* qkv; long long ld;        // a row: q heads x head_dim | k heads x head_dim | v heads x v_dim
  int n_tokens, n_heads, n_kv_heads, head_dim, v_dim;
  const float* q_norm_w; const float* k_norm_w; float eps;
  const float* cos_table; const float* sin_table; int rotary_dim, table_rows, interleaved;
  int v_unit_norm;
  const float* v_cos; const float* v_sin; int v_rotary_dim, v_table_rows, v_interleaved;
  const int* token_seq; const int* token_pos; const int* seq_slot; const int* seq_qstart;
  const int* page_table; int table_stride, num_pages;
  void* k_pages; void* v_pages;   // [num_pages, n_kv_heads, 64, head_dim] and [.., v_dim]
  int write_cache;
  int* status;
  const float* bias;   // [q | k | v features] added to the projected rows first (null: none)
  int qk_unit;         // != 0: q and k are divided by their root mean square over the head after the rotation
  // Values mixed with another layer's values of the same tokens: v <- (1 - v_lambda) v + v_lambda v_mix, before
  // anything else but the bias.  v_keep: the (mixed) values are also left there, for layers further on.
  const void* v_mix; void* v_keep;   // [n_tokens, n_kv_heads * v_dim] run dtype, or null
  float v_lambda;
};

template <typename T>
__global__ void qkv_rotate_append_kernel(QkvRotateArgs a) {
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y * (blockDim.x >> 5) + warp;
  const int total_heads = a.n_heads + 2 * a.n_kv_heads;
  const bool valid = t < a.n_tokens && head < total_heads;
  const bool is_q = head < a.n_heads;
  const bool is_k = !is_q && head < a.n_heads + a.n_kv_heads;
  const bool is_v = !is_q && !is_k;
  const int kv_head = is_q ? -1 : (is_k ? head - a.n_heads : head - a.n_heads - a.n_kv_heads);
  const int D = is_v ? a.v_dim : a.head_dim;
  const bool to_cache = valid && !is_q && a.write_cache;
  // the batch description and the page table do not come from the kernel before this one
  int pos = 0, seq = 0, slot = 0, q_begin = 0, q_end = 0, page = -1;
  if (valid) pos = a.token_pos[t];
  if (to_cache) {
    seq = a.token_seq[t];
    slot = a.seq_slot[seq];
    q_begin = a.seq_qstart[seq];
    q_end = a.seq_qstart[seq + 1];
    if (pos >= 0 && pos / kPageTokens < a.table_stride)
      page = a.page_table[(size_t)slot * a.table_stride + pos / kPageTokens];
  }
  pdl_wait_block();
  pdl_launch_dependents();
  if (!valid) return;
  const size_t row_off = is_v ? (size_t)(a.n_heads + a.n_kv_heads) * a.head_dim + (size_t)kv_head * a.v_dim
                              : (size_t)head * a.head_dim;
  T* row = (T*)a.qkv + (size_t)t * a.ld + row_off;
  T* cache_row = nullptr;
  if (to_cache) {
    if (pos < 0 || pos / kPageTokens >= a.table_stride) {
      if (lane == 0) report(a.status, kStatusPositionOutOfRange, t, pos, a.table_stride * kPageTokens);
    } else if (page < 0 || page >= a.num_pages) {
      if (lane == 0) report(a.status, kStatusPageOutOfRange, t, page, a.num_pages);
    } else {
      T* base = (T*)(is_k ? a.k_pages : a.v_pages);
      const int off = pos % kPageTokens;
      cache_row = base + (((size_t)page * a.n_kv_heads + kv_head) * kPageTokens + off) * D;
      // rows of a page beyond the sequence's last key must hold finite values (see the kernel above)
      if (t + 1 == q_end && off + 1 < kPageTokens && (off == 0 || q_end - q_begin > 1)) {
        T* rest = cache_row + D;
        const size_t n = (size_t)(kPageTokens - 1 - off) * D;
        for (size_t i = lane; i < n; i += 32) rest[i] = from_f32<T>(0.f);
      }
    }
  }
  const float* w = is_q ? a.q_norm_w : (is_k ? a.k_norm_w : nullptr);
  const bool normed = is_v ? (a.v_unit_norm != 0) : (w != nullptr);
  const float* bias = a.bias ? a.bias + row_off : nullptr;
  float inv = 1.f;
  if (normed) {
    float ss = 0.f;
    for (int c = lane; c < D; c += 32) {
      const float x = to_f32<T>(row[c]) + (bias ? bias[c] : 0.f);
      ss += x * x;
    }
    inv = rsqrtf(warp_sum(ss) / (float)D + a.eps);     // (values with a norm are not mixed: the launcher refuses that)
  }
  const float* ct = is_v ? a.v_cos : a.cos_table;
  const float* st = is_v ? a.v_sin : a.sin_table;
  const int rot = ct ? (is_v ? a.v_rotary_dim : a.rotary_dim) : 0;
  const int rows = is_v ? a.v_table_rows : a.table_rows;
  const bool inter = (is_v ? a.v_interleaved : a.interleaved) != 0;
  const int half = rot / 2;
  if (rot > 0 && (pos < 0 || pos >= rows)) {
    if (lane == 0) report(a.status, kStatusPositionOutOfRange, t, pos, rows);
    return;
  }
  const size_t v_off = is_v ? ((size_t)t * a.n_kv_heads + kv_head) * a.v_dim : 0;
  const T* v_mix = is_v && a.v_mix ? (const T*)a.v_mix + v_off : nullptr;
  T* v_keep = is_v && a.v_keep ? (T*)a.v_keep + v_off : nullptr;
  auto value = [&](int c) -> float {
    float x = to_f32<T>(row[c]);
    if (bias) x += bias[c];
    if (v_mix) x = (1.f - a.v_lambda) * x + a.v_lambda * to_f32<T>(v_mix[c]);
    if (normed) x *= inv;
    if (w) x *= w[c];
    return x;
  };
  float unit = 1.f;    // what the rotated q or k row is multiplied by
  auto put = [&](int c, float x) {
    const T o = from_f32<T>(x * unit);
    if (!is_v) row[c] = o;
    if (v_keep) v_keep[c] = o;
    if (cache_row) cache_row[c] = o;
  };
  auto turned = [&](int j, int& i0, int& i1, float& y0, float& y1) {
    i0 = inter ? 2 * j : j;
    i1 = inter ? 2 * j + 1 : j + half;
    const float x0 = value(i0), x1 = value(i1);
    const float c = ct[(size_t)pos * half + j], s = st[(size_t)pos * half + j];
    y0 = x0 * c - x1 * s;
    y1 = x1 * c + x0 * s;
  };
  int i0, i1;
  float y0, y1;
  if (a.qk_unit && !is_v) {
    float ss = 0.f;
    for (int j = lane; j < half; j += 32) {
      turned(j, i0, i1, y0, y1);
      ss += y0 * y0 + y1 * y1;
    }
    for (int c = rot + lane; c < D; c += 32) {
      const float x = value(c);
      ss += x * x;
    }
    unit = rsqrtf(warp_sum(ss) / (float)D + a.eps);
  }
  for (int j = lane; j < half; j += 32) {
    turned(j, i0, i1, y0, y1);
    put(i0, y0);
    put(i1, y1);
  }
  for (int c = rot + lane; c < D; c += 32) put(c, value(c));
}

// The general form for bfloat16 rows with 16-byte accesses and split-half pairs: bias, unit q and k after the rotation, mixed
// and kept values.  Head and value sizes of their own, multiples of 8 up to 256; half the rotated size a multiple of 8.
// A head takes size / 8 lanes (a warp holds as many whole heads as fit); a block's first warps take q and k heads, the rest
// values.  The lane that holds features [8i, 8i + 8) of the first rotated half trades its values with the lane that holds
// the matching features of the second half.  A block takes TPB tokens and has all their rows in flight before the first use.
template <int TPB>
__global__ void __launch_bounds__(256, TPB > 1 ? 5 : 1) qkv_rotate_append_halves_kernel(QkvRotateArgs a, int qk_warps) {
  typedef __nv_bfloat16 T;
  const int lane = threadIdx.x & 31;
  const int gw = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const bool is_v = gw >= qk_warps;
  const int D = is_v ? a.v_dim : a.head_dim;
  const int lph = D >> 3, per_warp = 32 / lph;
  const int sub = lane / lph, li = lane - sub * lph;
  const int idx = (is_v ? gw - qk_warps : gw) * per_warp + sub;       // head among q|k, or value head
  const bool active = sub < per_warp && idx < (is_v ? a.n_kv_heads : a.n_heads + a.n_kv_heads);
  const bool is_q = !is_v && idx < a.n_heads;
  const bool to_cache = active && !is_q && a.write_cache;
  const int kv_head = is_v ? idx : idx - a.n_heads;
  const int row_off = (is_v ? (a.n_heads + a.n_kv_heads) * a.head_dim + idx * D : idx * D) + 8 * li;
  const int t0 = blockIdx.x * TPB;
  // the batch description and the page table do not come from the kernel before this one; with one token a block they are
  // fetched while it may still run
  int pos0 = 0, page0 = -1, seq0 = 0;
  auto find_page = [&](int t, int pos) -> int {
    if (pos < 0 || pos / kPageTokens >= a.table_stride) return -1;
    return a.page_table[(size_t)a.seq_slot[a.token_seq[t]] * a.table_stride + pos / kPageTokens];
  };
  if (TPB == 1 && t0 < a.n_tokens) {
    pos0 = a.token_pos[t0];
    if (to_cache) {
      page0 = find_page(t0, pos0);
      seq0 = a.token_seq[t0];
    }
  }
  float bv[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) bv[e] = 0.f;
  if (active && a.bias) {
    const float4 b0 = *reinterpret_cast<const float4*>(a.bias + row_off), b1 = *reinterpret_cast<const float4*>(a.bias + row_off + 4);
    bv[0] = b0.x; bv[1] = b0.y; bv[2] = b0.z; bv[3] = b0.w; bv[4] = b1.x; bv[5] = b1.y; bv[6] = b1.z; bv[7] = b1.w;
  }
  pdl_wait_block();
  pdl_launch_dependents();
  auto unpack = [&](const uint4& raw, float (&x)[8]) {
    const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(h2[e]);
      x[2 * e] = f.x;
      x[2 * e + 1] = f.y;
    }
  };
  // where this lane's piece of token t goes in the cache (null: nowhere); clears the rest of a page where the first kernel does
  auto cache_place = [&](int t, int pos, int page) -> T* {
    if (!to_cache) return nullptr;
    if (pos < 0 || pos / kPageTokens >= a.table_stride) {
      if (li == 0) report(a.status, kStatusPositionOutOfRange, t, pos, a.table_stride * kPageTokens);
      return nullptr;
    }
    if (page < 0 || page >= a.num_pages) {
      if (li == 0) report(a.status, kStatusPageOutOfRange, t, page, a.num_pages);
      return nullptr;
    }
    const int off = pos % kPageTokens;
    T* head_row = (T*)(is_v ? a.v_pages : a.k_pages) + (((size_t)page * a.n_kv_heads + kv_head) * kPageTokens + off) * D;
    const int b = TPB == 1 ? seq0 : a.token_seq[t];
    const int q_end = a.seq_qstart[b + 1];
    if (t + 1 == q_end && off + 1 < kPageTokens && (off == 0 || q_end - a.seq_qstart[b] > 1)) {
      uint4* r4 = reinterpret_cast<uint4*>(head_row + D);
      const int n4 = (kPageTokens - 1 - off) * D / 8;
      for (int x = li; x < n4; x += lph) r4[x] = make_uint4(0, 0, 0, 0);
    }
    return head_row + 8 * li;
  };
  auto pack = [&](const float (&x)[8]) -> uint4 {
    uint4 out;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
    for (int e = 0; e < 4; ++e) o2[e] = __floats2bfloat162_rn(x[2 * e], x[2 * e + 1]);
    return out;
  };
  uint4 raws[TPB];
  int poss[TPB], pages[TPB];
#pragma unroll
  for (int i = 0; i < TPB; ++i) {
    const int t = t0 + i;
    raws[i] = make_uint4(0, 0, 0, 0);
    poss[i] = pos0;
    pages[i] = page0;
    if (t < a.n_tokens) {
      if (active) raws[i] = *reinterpret_cast<const uint4*>((const T*)a.qkv + (size_t)t * a.ld + row_off);
      if (TPB > 1) {
        poss[i] = a.token_pos[t];
        if (to_cache) pages[i] = find_page(t, poss[i]);
      }
    }
  }
  if (is_v) {                               // (whole warps: nothing below shuffles across q|k and value warps)
    const size_t v_off = (size_t)idx * D + 8 * li;
    uint4 mixed[TPB];
#pragma unroll
    for (int i = 0; i < TPB; ++i) {
      mixed[i] = make_uint4(0, 0, 0, 0);
      if (active && a.v_mix && t0 + i < a.n_tokens)
        mixed[i] = *reinterpret_cast<const uint4*>((const T*)a.v_mix + (size_t)(t0 + i) * a.n_kv_heads * D + v_off);
    }
    if (!active) return;
#pragma unroll
    for (int i = 0; i < TPB; ++i) {
      const int t = t0 + i;
      if (t >= a.n_tokens) break;
      T* cache_row = cache_place(t, poss[i], pages[i]);
      float x[8], f[8];
      unpack(raws[i], x);
      unpack(mixed[i], f);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        x[e] += bv[e];
        if (a.v_mix) x[e] = (1.f - a.v_lambda) * x[e] + a.v_lambda * f[e];
      }
      const uint4 out = pack(x);
      if (a.v_keep) *reinterpret_cast<uint4*>((T*)a.v_keep + (size_t)t * a.n_kv_heads * D + v_off) = out;
      if (cache_row) *reinterpret_cast<uint4*>(cache_row) = out;
    }
    return;
  }
  const int rot = a.rotary_dim, half = rot >> 1, half_l = half >> 3;
  const bool turns = active && 8 * li < rot;
  const bool second = li >= half_l;
  const int j = 8 * (second ? li - half_l : li);
  const int partner = (turns ? lane + (second ? -half_l : half_l) : lane) & 31;
  const float sign = second ? 1.f : -1.f;
  const bool pow2 = (lph & (lph - 1)) == 0;
#pragma unroll
  for (int i = 0; i < TPB; ++i) {
    const int t = t0 + i;
    if (t >= a.n_tokens) break;
    const int pos = poss[i];
    float x[8];
    unpack(raws[i], x);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] += bv[e];
    bool ok = true;
    if (rot > 0) {
      ok = !turns || (pos >= 0 && pos < a.table_rows);
      if (!ok && li == 0) report(a.status, kStatusPositionOutOfRange, t, pos, a.table_rows);
      const size_t at = (size_t)(turns && ok ? pos : 0) * half + (turns ? j : 0);
#pragma unroll
      for (int h = 0; h < 2; ++h) {        // the tables stay in L2
        const float4 c = *reinterpret_cast<const float4*>(a.cos_table + at + 4 * h), s = *reinterpret_cast<const float4*>(a.sin_table + at + 4 * h);
        const float cv[4] = {c.x, c.y, c.z, c.w}, sv[4] = {s.x, s.y, s.z, s.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float other = __shfl_sync(0xffffffffu, x[4 * h + e], partner);
          const float y = fmaf(sign * sv[e], other, x[4 * h + e] * cv[e]);
          x[4 * h + e] = turns ? y : x[4 * h + e];
        }
      }
    }
    if (a.qk_unit) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
      if (pow2) {
        for (int o = lph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      } else {
        float total = 0.f;
        for (int l = 0; l < lph; ++l) total += __shfl_sync(0xffffffffu, ss, (sub * lph + l) & 31);
        ss = total;
      }
      const float inv = rsqrtf(ss / (float)D + a.eps);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] *= inv;
    }
    T* cache_row = cache_place(t, pos, pages[i]);
    if (!active || !ok) continue;
    const uint4 out = pack(x);
    *reinterpret_cast<uint4*>((T*)a.qkv + (size_t)t * a.ld + row_off) = out;
    if (cache_row) *reinterpret_cast<uint4*>(cache_row) = out;
  }
}

// The general form for bfloat16 rows with 16-byte accesses: keys and values of one size that is a multiple of 8 (up to
// 256), interleaved pairs, rotated sizes that are multiples of 8, everything 16-byte aligned.  A head takes
// head_dim / 8 lanes; a lane's eight features are four whole pairs, so the rotation needs no other lane.  A block takes
// TPB tokens and has all their rows and positions in flight before it uses the first.
template <int TPB>
__global__ void __launch_bounds__(256, 4) qkv_rotate_append_vec8_kernel(QkvRotateArgs a, int lanes_per_head) {
  pdl_wait_block();
  pdl_launch_dependents();
  typedef __nv_bfloat16 T;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int lph = lanes_per_head, heads_per_warp = 32 / lph;
  const int sub = lane / lph, li = lane - sub * lph;
  const int total_heads = a.n_heads + 2 * a.n_kv_heads;
  const int head = (blockIdx.y * (blockDim.x >> 5) + warp) * heads_per_warp + sub;
  const bool active = sub < heads_per_warp && head < total_heads;
  const int d = a.head_dim;
  const bool is_q = head < a.n_heads;
  const bool is_k = !is_q && head < a.n_heads + a.n_kv_heads;
  const bool is_v = !is_q && !is_k;
  const int kv_head = is_k ? head - a.n_heads : head - a.n_heads - a.n_kv_heads;
  const bool pow2 = (lph & (lph - 1)) == 0;
  const float* w = is_q ? a.q_norm_w : (is_k ? a.k_norm_w : nullptr);
  const bool normed = is_v ? (a.v_unit_norm != 0) : (w != nullptr);
  const float* ct = is_v ? a.v_cos : a.cos_table;
  const float* st = is_v ? a.v_sin : a.sin_table;
  const int rot = ct ? (is_v ? a.v_rotary_dim : a.rotary_dim) : 0;
  const int rows = is_v ? a.v_table_rows : a.table_rows;
  const int half = rot / 2;
  const bool turns = active && 8 * li < rot;
  float wv[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) wv[e] = 1.f;
  if (active && w) {
    const float4 w0 = *reinterpret_cast<const float4*>(w + 8 * li), w1 = *reinterpret_cast<const float4*>(w + 8 * li + 4);
    wv[0] = w0.x; wv[1] = w0.y; wv[2] = w0.z; wv[3] = w0.w; wv[4] = w1.x; wv[5] = w1.y; wv[6] = w1.z; wv[7] = w1.w;
  }
  uint4 raws[TPB];
  int poss[TPB];
#pragma unroll
  for (int i = 0; i < TPB; ++i) {
    const int t = blockIdx.x * TPB + i;
    raws[i] = make_uint4(0, 0, 0, 0);
    poss[i] = -1;
    if (t < a.n_tokens) {
      if (active) raws[i] = *reinterpret_cast<const uint4*>((const T*)a.qkv + (size_t)t * a.ld + (size_t)head * d + 8 * li);
      poss[i] = a.token_pos[t];
    }
  }
#pragma unroll
  for (int i = 0; i < TPB; ++i) {
    const int t = blockIdx.x * TPB + i;
    if (t >= a.n_tokens) break;
    T* row = (T*)a.qkv + (size_t)t * a.ld + (size_t)head * d + 8 * li;
    const int pos = poss[i];
    T* cache_row = nullptr;
    if (active && !is_q && a.write_cache) {
      const int b = a.token_seq[t];
      const int slot = a.seq_slot[b];
      const int logical = pos / kPageTokens;
      if (pos < 0 || logical >= a.table_stride) {
        if (li == 0) report(a.status, kStatusPositionOutOfRange, t, pos, a.table_stride * kPageTokens);
      } else {
        const int page = a.page_table[(size_t)slot * a.table_stride + logical];
        if (page < 0 || page >= a.num_pages) {
          if (li == 0) report(a.status, kStatusPageOutOfRange, t, page, a.num_pages);
        } else {
          T* base = (T*)(is_k ? a.k_pages : a.v_pages);
          const int off = pos % kPageTokens;
          T* head_row = base + (((size_t)page * a.n_kv_heads + kv_head) * kPageTokens + off) * d;
          cache_row = head_row + 8 * li;
          const int q_end = a.seq_qstart[b + 1];
          if (t + 1 == q_end && off + 1 < kPageTokens && (off == 0 || q_end - a.seq_qstart[b] > 1)) {
            uint4* r4 = reinterpret_cast<uint4*>(head_row + d);      // clear the rest of the page (see the first kernel)
            const size_t n4 = (size_t)(kPageTokens - 1 - off) * d / 8;
            for (size_t x = li; x < n4; x += lph) r4[x] = make_uint4(0, 0, 0, 0);
          }
        }
      }
    }
    float x[8];
    {
      const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raws[i]);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(h2[e]);
        x[2 * e] = f.x;
        x[2 * e + 1] = f.y;
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
    if (pow2) {
      for (int o = lph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    } else {
      float total = 0.f;
      for (int l = 0; l < lph; ++l) total += __shfl_sync(0xffffffffu, ss, (sub * lph + l) & 31);
      ss = total;
    }
    if (!active) continue;
    if (normed) {
      const float inv = rsqrtf(ss / (float)d + a.eps);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] = x[e] * inv * wv[e];
    }
    if (turns) {
      if (pos < 0 || pos >= rows) {
        if (li == 0) report(a.status, kStatusPositionOutOfRange, t, pos, rows);
        continue;
      }
      const float4 c4 = *reinterpret_cast<const float4*>(ct + (size_t)pos * half + 4 * li);
      const float4 s4 = *reinterpret_cast<const float4*>(st + (size_t)pos * half + 4 * li);
      const float cc[4] = {c4.x, c4.y, c4.z, c4.w}, sn[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float x0 = x[2 * e], x1 = x[2 * e + 1];
        x[2 * e] = x0 * cc[e] - x1 * sn[e];
        x[2 * e + 1] = x1 * cc[e] + x0 * sn[e];
      }
    }
    uint4 out;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
    for (int e = 0; e < 4; ++e) o2[e] = __floats2bfloat162_rn(x[2 * e], x[2 * e + 1]);
    if (!is_v) *reinterpret_cast<uint4*>(row) = out;
    if (cache_row) *reinterpret_cast<uint4*>(cache_row) = out;
  }
}

// ---- one norm over all heads ------------------------------------------------------------------------------------
// The form in which q and k are each divided by the root mean square of the whole projection (all heads together) and
// multiplied by a weight of that length; queries may carry a temperature that grows with their position:
//   q <- unit(q_row) * w_q * (1 + coef * ln(floor((p + 1) / every) + 1)) ;  k <- unit(k_row) * w_k
// then the rotation (either layout of pairs, or none) and the append as above; values go to the cache as they are.  Without
// weights nothing is divided.  One block per token; the row's two sums meet in shared memory before anything is written.
struct QkvRowArgs {
  QkvRotateArgs r;
  float temp_coef; int temp_every;   // temp_every <= 0: no temperature
};

__device__ __forceinline__ float query_temperature(const QkvRowArgs& a, int pos) {
  if (a.temp_every <= 0) return 1.f;
  return fmaf(a.temp_coef, logf((float)((pos + 1) / a.temp_every) + 1.f), 1.f);
}

// The page that holds position `pos` of token t's sequence; -1 (with a report by the first thread) if there is none.
__device__ __forceinline__ int row_page(const QkvRotateArgs& a, int t, int pos) {
  if (pos < 0 || pos / kPageTokens >= a.table_stride) {
    if (threadIdx.x == 0) report(a.status, kStatusPositionOutOfRange, t, pos, a.table_stride * kPageTokens);
    return -1;
  }
  const int page = a.page_table[(size_t)a.seq_slot[a.token_seq[t]] * a.table_stride + pos / kPageTokens];
  if (page < 0 || page >= a.num_pages) {
    if (threadIdx.x == 0) report(a.status, kStatusPageOutOfRange, t, page, a.num_pages);
    return -1;
  }
  return page;
}

// Whether token t clears the rows of its page behind its own (see the first kernel for when and why).
__device__ __forceinline__ bool clears_page(const QkvRotateArgs& a, int t, int off) {
  const int b = a.token_seq[t], q_begin = a.seq_qstart[b], q_end = a.seq_qstart[b + 1];
  return t + 1 == q_end && off + 1 < kPageTokens && (off == 0 || q_end - q_begin > 1);
}

template <typename T>
__global__ void __launch_bounds__(256) qkv_row_norm_append_kernel(QkvRowArgs x) {
  __shared__ float red[32];
  const QkvRotateArgs& a = x.r;
  const int t = blockIdx.x;
  // the batch description and the page table do not come from the kernel before this one
  const int pos = a.token_pos[t];
  const int page = a.write_cache ? row_page(a, t, pos) : -1;
  const int off = pos % kPageTokens;
  const bool clears = page >= 0 && clears_page(a, t, off);
  pdl_wait_block();
  pdl_launch_dependents();
  const int d = a.head_dim, dv = a.v_dim, H = a.n_heads, G = a.n_kv_heads;
  T* row = (T*)a.qkv + (size_t)t * a.ld;
  const int q_cols = H * d, k_cols = G * d;
  float inv_q = 1.f, inv_k = 1.f;
  if (a.q_norm_w) {
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x; c < q_cols; c += blockDim.x) {
      const float v = to_f32<T>(row[c]);
      sq = fmaf(v, v, sq);
    }
    for (int c = threadIdx.x; c < k_cols; c += blockDim.x) {
      const float v = to_f32<T>(row[q_cols + c]);
      sk = fmaf(v, v, sk);
    }
    inv_q = rsqrtf(block_sum(sq, red) / (float)q_cols + a.eps);
    inv_k = rsqrtf(block_sum(sk, red) / (float)k_cols + a.eps);
  }
  const int rot = a.cos_table ? a.rotary_dim : 0, half = rot / 2;
  if (rot > 0 && (pos < 0 || pos >= a.table_rows)) {
    if (threadIdx.x == 0) report(a.status, kStatusPositionOutOfRange, t, pos, a.table_rows);
    return;
  }
  inv_q *= query_temperature(x, pos);
  auto value = [&](int head, int c) -> float {
    const bool is_q = head < H;
    const int col = head * d + c;
    float v = to_f32<T>(row[col]) * (is_q ? inv_q : inv_k);
    if (a.q_norm_w) v *= is_q ? a.q_norm_w[col] : a.k_norm_w[col - q_cols];
    return v;
  };
  auto put = [&](int head, int c, float v) {
    const T o = from_f32<T>(v);
    if (head < H) row[head * d + c] = o;
    else if (page >= 0) ((T*)a.k_pages)[(((size_t)page * G + (head - H)) * kPageTokens + off) * d + c] = o;
  };
  const int units = half + (d - rot);      // pairs, then single features
  for (int i = threadIdx.x; i < (H + G) * units; i += blockDim.x) {
    const int head = i / units, u = i - head * units;
    if (u < half) {
      const int i0 = a.interleaved ? 2 * u : u, i1 = a.interleaved ? 2 * u + 1 : u + half;
      const float x0 = value(head, i0), x1 = value(head, i1);
      const float c = a.cos_table[(size_t)pos * half + u], s = a.sin_table[(size_t)pos * half + u];
      put(head, i0, x0 * c - x1 * s);
      put(head, i1, x1 * c + x0 * s);
    } else {
      const int c = rot + (u - half);
      put(head, c, value(head, c));
    }
  }
  if (page < 0) return;
  const T* v_row = row + q_cols + k_cols;
  for (int i = threadIdx.x; i < G * dv; i += blockDim.x) {
    const int g = i / dv, c = i - g * dv;
    ((T*)a.v_pages)[(((size_t)page * G + g) * kPageTokens + off) * dv + c] = v_row[i];
  }
  if (clears) {
    const int rest = kPageTokens - 1 - off;
    for (int g = 0; g < G; ++g) {
      const size_t first = ((size_t)page * G + g) * kPageTokens + off + 1;
      for (int i = threadIdx.x; i < rest * d; i += blockDim.x) ((T*)a.k_pages)[first * d + i] = from_f32<T>(0.f);
      for (int i = threadIdx.x; i < rest * dv; i += blockDim.x) ((T*)a.v_pages)[first * dv + i] = from_f32<T>(0.f);
    }
  }
}

// The same for bfloat16 rows without a rotation, 16 bytes an access (head sizes multiples of 8, everything 16-byte aligned): a
// thread holds up to VPT pieces of the row in registers, all in flight before the first use.
template <int VPT>
__global__ void __launch_bounds__(1024) qkv_row_norm_append_vec8_kernel(QkvRowArgs x) {
  typedef __nv_bfloat16 T;
  __shared__ float red_q[32], red_k[32];
  const QkvRotateArgs& a = x.r;
  const int t = blockIdx.x;
  const int pos = a.token_pos[t];
  const int page = a.write_cache ? row_page(a, t, pos) : -1;
  const int off = pos % kPageTokens;
  const bool clears = page >= 0 && clears_page(a, t, off);
  const int d8 = a.head_dim / 8, dv8 = a.v_dim / 8, G = a.n_kv_heads;
  const int q8 = a.n_heads * d8, k8 = q8 + G * d8, all8 = k8 + G * dv8;
  const float temp = query_temperature(x, pos);
  pdl_wait_block();
  pdl_launch_dependents();
  uint4* row = reinterpret_cast<uint4*>((T*)a.qkv + (size_t)t * a.ld);
  uint4 raw[VPT];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    raw[k] = i < all8 ? row[i] : make_uint4(0, 0, 0, 0);
  }
  float inv_q = 1.f, inv_k = 1.f;
  if (a.q_norm_w) {
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = threadIdx.x + k * blockDim.x;
      const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw[k]);
      float s = 0.f;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(h2[e]);
        s = fmaf(f.x, f.x, fmaf(f.y, f.y, s));
      }
      if (i < q8) sq += s;
      else if (i < k8) sk += s;
    }
    // both sums at one barrier
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = (blockDim.x + 31) >> 5;
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) { red_q[warp] = sq; red_k[warp] = sk; }
    __syncthreads();
    sq = warp_sum(lane < n_warps ? red_q[lane] : 0.f);
    sk = warp_sum(lane < n_warps ? red_k[lane] : 0.f);
    inv_q = rsqrtf(sq / (float)(q8 * 8) + a.eps);
    inv_k = rsqrtf(sk / (float)((k8 - q8) * 8) + a.eps);
  }
  inv_q *= temp;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i >= all8) break;
    if (i >= k8) {                         // a value: to its page as it is
      if (page < 0) continue;
      const int j = i - k8, g = j / dv8, c = j - g * dv8;
      reinterpret_cast<uint4*>(a.v_pages)[(((size_t)page * G + g) * kPageTokens + off) * dv8 + c] = raw[k];
      continue;
    }
    const bool is_q = i < q8;
    const float inv = is_q ? inv_q : inv_k;
    float f[8];
    const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw[k]);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 v = __bfloat1622float2(h2[e]);
      f[2 * e] = v.x * inv;
      f[2 * e + 1] = v.y * inv;
    }
    if (a.q_norm_w) {
      const float4* w = reinterpret_cast<const float4*>(is_q ? a.q_norm_w + 8 * i : a.k_norm_w + 8 * (i - q8));
      const float4 w0 = w[0], w1 = w[1];
      f[0] *= w0.x; f[1] *= w0.y; f[2] *= w0.z; f[3] *= w0.w; f[4] *= w1.x; f[5] *= w1.y; f[6] *= w1.z; f[7] *= w1.w;
    }
    uint4 out;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
    for (int e = 0; e < 4; ++e) o2[e] = __floats2bfloat162_rn(f[2 * e], f[2 * e + 1]);
    if (is_q) {
      row[i] = out;
    } else if (page >= 0) {
      const int j = i - q8, g = j / d8, c = j - g * d8;
      reinterpret_cast<uint4*>(a.k_pages)[(((size_t)page * G + g) * kPageTokens + off) * d8 + c] = out;
    }
  }
  if (clears) {
    const int rest = kPageTokens - 1 - off;
    for (int g = 0; g < G; ++g) {
      const size_t first = ((size_t)page * G + g) * kPageTokens + off + 1;
      for (int i = threadIdx.x; i < rest * d8; i += blockDim.x) reinterpret_cast<uint4*>(a.k_pages)[first * d8 + i] = make_uint4(0, 0, 0, 0);
      for (int i = threadIdx.x; i < rest * dv8; i += blockDim.x) reinterpret_cast<uint4*>(a.v_pages)[first * dv8 + i] = make_uint4(0, 0, 0, 0);
    }
  }
}

}  // namespace pe

extern "C" int pe_batch_expand(const int* seq_qstart, const int* seq_past, int n_seqs, int* token_seq, int* token_pos,
                               cudaStream_t stream) {
  if (n_seqs <= 0) return PE_OK;
  pe::launch(pe::batch_expand_kernel, n_seqs, 128, 0, stream, seq_qstart, seq_past, n_seqs, token_seq, token_pos);
  PE_LAUNCH_CHECK();
  return PE_OK;
}

extern "C" int pe_qk_norm_rope_append(int dtype, void* qkv, long long ld, int n_tokens, int n_heads, int n_kv_heads,
                                      int head_dim, const float* q_norm_w, const float* k_norm_w, float eps,
                                      const float* cos_table, const float* sin_table, int rotary_dim, int table_rows,
                                      const int* token_seq, const int* token_pos, const int* seq_slot,
                                      const int* seq_qstart, const int* page_table, int table_stride, int num_pages, void* k_pages,
                                      void* v_pages, int write_cache, int* status, cudaStream_t stream) {
  if (n_tokens <= 0) return PE_OK;
  if (head_dim <= 0 || n_heads <= 0 || n_kv_heads < 0) return PE_ERR_BAD_ARGUMENT;
  if (rotary_dim < 0 || rotary_dim > head_dim || (rotary_dim & 1)) return PE_ERR_UNSUPPORTED_SIZE;
  if (ld < (long long)(n_heads + 2 * n_kv_heads) * head_dim) return PE_ERR_BAD_ARGUMENT;
  pe::RopeAppendArgs a;
  a.qkv = qkv; a.ld = ld; a.n_tokens = n_tokens; a.n_heads = n_heads; a.n_kv_heads = n_kv_heads; a.head_dim = head_dim;
  a.q_norm_w = q_norm_w; a.k_norm_w = k_norm_w; a.eps = eps;
  a.cos_table = cos_table; a.sin_table = sin_table; a.rotary_dim = rotary_dim; a.table_rows = table_rows;
  a.token_seq = token_seq; a.token_pos = token_pos; a.seq_slot = seq_slot; a.seq_qstart = seq_qstart;
  a.page_table = page_table; a.table_stride = table_stride; a.num_pages = num_pages;
  a.k_pages = k_pages; a.v_pages = v_pages; a.write_cache = write_cache; a.status = status;
  const int warps = 4;
  const int total_heads = n_heads + 2 * n_kv_heads;
  dim3 grid(n_tokens, (total_heads + warps - 1) / warps);
  if (grid.y > 65535) return PE_ERR_UNSUPPORTED_SIZE;
  // two features per access where everything is even and aligned (the usual case)
  const size_t esz = dtype == PE_F32 ? 4 : 2;
  const bool pairs = (head_dim % 2 == 0) && (rotary_dim % 4 == 0) && (ld % 2 == 0) && ((uintptr_t)qkv % (2 * esz) == 0) &&
                     ((uintptr_t)k_pages % (2 * esz) == 0) && ((uintptr_t)v_pages % (2 * esz) == 0) &&
                     ((uintptr_t)cos_table % 8 == 0) && ((uintptr_t)sin_table % 8 == 0) &&
                     ((uintptr_t)q_norm_w % 8 == 0) && ((uintptr_t)k_norm_w % 8 == 0);
  const bool vec8 = dtype == PE_BF16 && head_dim % 16 == 0 && head_dim <= 256 && (rotary_dim == head_dim || cos_table == nullptr) &&
                    ld % 8 == 0 && (uintptr_t)qkv % 16 == 0 && (uintptr_t)k_pages % 16 == 0 && (uintptr_t)v_pages % 16 == 0 &&
                    (uintptr_t)cos_table % 16 == 0 && (uintptr_t)sin_table % 16 == 0 && (uintptr_t)q_norm_w % 16 == 0 &&
                    (uintptr_t)k_norm_w % 16 == 0;
  if (vec8 && n_tokens >= 256) {  // measured: with a few tokens (decode) the kernel above is the faster one
    constexpr int kTokensPerBlock = 4;
    const int lph = head_dim / 8, heads_per_block = 8 * (32 / lph);
    dim3 g((n_tokens + kTokensPerBlock - 1) / kTokensPerBlock, (total_heads + heads_per_block - 1) / heads_per_block);
    if (g.y > 65535) return PE_ERR_UNSUPPORTED_SIZE;
    pe::launch(pe::qk_norm_rope_append_vec8_kernel<kTokensPerBlock>, g, 256, 0, stream, a, lph);
    PE_LAUNCH_CHECK();
    return PE_OK;
  }
  if (dtype == PE_F32) {
    if (pairs) pe::launch(pe::qk_norm_rope_append_kernel<float, true>, grid, warps * 32, 0, stream, a);
    else pe::launch(pe::qk_norm_rope_append_kernel<float, false>, grid, warps * 32, 0, stream, a);
  } else if (dtype == PE_BF16) {
    if (pairs) pe::launch(pe::qk_norm_rope_append_kernel<__nv_bfloat16, true>, grid, warps * 32, 0, stream, a);
    else pe::launch(pe::qk_norm_rope_append_kernel<__nv_bfloat16, false>, grid, warps * 32, 0, stream, a);
  } else
    return PE_ERR_UNSUPPORTED_DTYPE;
  PE_LAUNCH_CHECK();
  return PE_OK;
}

extern "C" int pe_qkv_rotate_append(int dtype, void* qkv, long long ld, int n_tokens, int n_heads, int n_kv_heads,
                                    int head_dim, int v_dim, const float* q_norm_w, const float* k_norm_w, float eps,
                                    const float* cos_table, const float* sin_table, int rotary_dim, int table_rows,
                                    int interleaved, int v_unit_norm, const float* v_cos, const float* v_sin,
                                    int v_rotary_dim, int v_table_rows, int v_interleaved, const int* token_seq,
                                    const int* token_pos, const int* seq_slot, const int* seq_qstart,
                                    const int* page_table, int table_stride, int num_pages, void* k_pages,
                                    void* v_pages, int write_cache, const float* bias, int qk_unit, const void* v_mix,
                                    float v_lambda, void* v_keep, int* status, cudaStream_t stream) {
  if (n_tokens <= 0) return PE_OK;
  if (v_mix && v_unit_norm) return PE_ERR_BAD_ARGUMENT;
  if (head_dim <= 0 || v_dim <= 0 || n_heads <= 0 || n_kv_heads < 0) return PE_ERR_BAD_ARGUMENT;
  if (rotary_dim < 0 || rotary_dim > head_dim || (rotary_dim & 1)) return PE_ERR_UNSUPPORTED_SIZE;
  if (v_rotary_dim < 0 || v_rotary_dim > v_dim || (v_rotary_dim & 1)) return PE_ERR_UNSUPPORTED_SIZE;
  if (ld < (long long)(n_heads + n_kv_heads) * head_dim + (long long)n_kv_heads * v_dim) return PE_ERR_BAD_ARGUMENT;
  pe::QkvRotateArgs a;
  a.qkv = qkv; a.ld = ld; a.n_tokens = n_tokens; a.n_heads = n_heads; a.n_kv_heads = n_kv_heads; a.head_dim = head_dim;
  a.v_dim = v_dim; a.q_norm_w = q_norm_w; a.k_norm_w = k_norm_w; a.eps = eps;
  a.cos_table = cos_table; a.sin_table = sin_table; a.rotary_dim = cos_table ? rotary_dim : 0; a.table_rows = table_rows;
  a.interleaved = interleaved; a.v_unit_norm = v_unit_norm;
  a.v_cos = v_cos; a.v_sin = v_sin; a.v_rotary_dim = v_cos ? v_rotary_dim : 0; a.v_table_rows = v_table_rows;
  a.v_interleaved = v_interleaved;
  a.token_seq = token_seq; a.token_pos = token_pos; a.seq_slot = seq_slot; a.seq_qstart = seq_qstart;
  a.page_table = page_table; a.table_stride = table_stride; a.num_pages = num_pages;
  a.k_pages = k_pages; a.v_pages = v_pages; a.write_cache = write_cache; a.status = status; a.bias = bias;
  a.qk_unit = qk_unit; a.v_mix = v_mix; a.v_keep = v_keep; a.v_lambda = v_lambda;
  const int warps = 4;
  dim3 grid(n_tokens, (n_heads + 2 * n_kv_heads + warps - 1) / warps);
  if (grid.y > 65535) return PE_ERR_UNSUPPORTED_SIZE;
  auto al16 = [](const void* p) { return (uintptr_t)p % 16 == 0; };
  const bool halves = dtype == PE_BF16 && q_norm_w == nullptr && k_norm_w == nullptr && !v_unit_norm && a.v_rotary_dim == 0 &&
                      head_dim % 8 == 0 && head_dim <= 256 && v_dim % 8 == 0 && v_dim <= 256 && ld % 8 == 0 &&
                      (a.rotary_dim == 0 || (!interleaved && a.rotary_dim % 16 == 0)) && al16(qkv) && al16(k_pages) && al16(v_pages) &&
                      al16(cos_table) && al16(sin_table) && al16(bias) && al16(v_mix) && al16(v_keep);
  if (halves) {
    const int qk_per_warp = 32 / (head_dim / 8), v_per_warp = 32 / (v_dim / 8);
    const int qk_warps = (n_heads + n_kv_heads + qk_per_warp - 1) / qk_per_warp;
    const int all_warps = qk_warps + (n_kv_heads + v_per_warp - 1) / v_per_warp;
    if (n_tokens >= 256) {
      constexpr int kTokensPerBlock = 2;   // (2,048 tokens, 16 + 4 heads of 128: 2 tokens 21.6 us, 3 23.8, 4 28.7, 8 38.0)
      dim3 g((n_tokens + kTokensPerBlock - 1) / kTokensPerBlock, (all_warps + 7) / 8);
      if (g.y > 65535) return PE_ERR_UNSUPPORTED_SIZE;
      pe::launch(pe::qkv_rotate_append_halves_kernel<kTokensPerBlock>, g, 256, 0, stream, a, qk_warps);
    } else {
      dim3 g(n_tokens, (all_warps + 3) / 4);
      if (g.y > 65535) return PE_ERR_UNSUPPORTED_SIZE;
      pe::launch(pe::qkv_rotate_append_halves_kernel<1>, g, 128, 0, stream, a, qk_warps);
    }
    PE_LAUNCH_CHECK();
    return PE_OK;
  }
  const bool vec8 = dtype == PE_BF16 && bias == nullptr && !qk_unit && !v_mix && !v_keep && head_dim == v_dim && head_dim % 8 == 0 && head_dim <= 256 && ld % 8 == 0 &&
                    (a.rotary_dim == 0 || (interleaved && a.rotary_dim % 8 == 0)) &&
                    (a.v_rotary_dim == 0 || (v_interleaved && a.v_rotary_dim % 8 == 0)) && al16(qkv) && al16(k_pages) &&
                    al16(v_pages) && al16(cos_table) && al16(sin_table) && al16(v_cos) && al16(v_sin) && al16(q_norm_w) &&
                    al16(k_norm_w);
  if (vec8 && n_tokens >= 256) {   // as for the kernel it stands beside: with a few tokens the one-warp-a-head form is faster
    constexpr int kTokensPerBlock = 4;
    const int lph = head_dim / 8, heads_per_block = 8 * (32 / lph);
    dim3 g((n_tokens + kTokensPerBlock - 1) / kTokensPerBlock, (n_heads + 2 * n_kv_heads + heads_per_block - 1) / heads_per_block);
    if (g.y > 65535) return PE_ERR_UNSUPPORTED_SIZE;
    pe::launch(pe::qkv_rotate_append_vec8_kernel<kTokensPerBlock>, g, 256, 0, stream, a, lph);
    PE_LAUNCH_CHECK();
    return PE_OK;
  }
  if (dtype == PE_F32) pe::launch(pe::qkv_rotate_append_kernel<float>, grid, warps * 32, 0, stream, a);
  else if (dtype == PE_BF16) pe::launch(pe::qkv_rotate_append_kernel<__nv_bfloat16>, grid, warps * 32, 0, stream, a);
  else return PE_ERR_UNSUPPORTED_DTYPE;
  PE_LAUNCH_CHECK();
  return PE_OK;
}

// q_norm_w [n_heads * head_dim] and k_norm_w [n_kv_heads * head_dim]: both or neither.  temp_every <= 0: no temperature.
extern "C" int pe_qkv_row_norm_append(int dtype, void* qkv, long long ld, int n_tokens, int n_heads, int n_kv_heads, int head_dim,
                                      int v_dim, const float* q_norm_w, const float* k_norm_w, float eps, float temp_coef,
                                      int temp_every, const float* cos_table, const float* sin_table, int rotary_dim,
                                      int table_rows, int interleaved, const int* token_seq, const int* token_pos,
                                      const int* seq_slot, const int* seq_qstart, const int* page_table, int table_stride,
                                      int num_pages, void* k_pages, void* v_pages, int write_cache, int* status,
                                      cudaStream_t stream) {
  if (n_tokens <= 0) return PE_OK;
  if (dtype != PE_F32 && dtype != PE_BF16) return PE_ERR_UNSUPPORTED_DTYPE;
  if (head_dim <= 0 || v_dim <= 0 || n_heads <= 0 || n_kv_heads <= 0) return PE_ERR_BAD_ARGUMENT;
  if ((q_norm_w == nullptr) != (k_norm_w == nullptr) || (cos_table == nullptr) != (sin_table == nullptr)) return PE_ERR_BAD_ARGUMENT;
  if (rotary_dim < 0 || rotary_dim > head_dim || (rotary_dim & 1)) return PE_ERR_UNSUPPORTED_SIZE;
  if (ld < (long long)(n_heads + n_kv_heads) * head_dim + (long long)n_kv_heads * v_dim) return PE_ERR_BAD_ARGUMENT;
  pe::QkvRowArgs x = {};
  pe::QkvRotateArgs& a = x.r;
  a.qkv = qkv; a.ld = ld; a.n_tokens = n_tokens; a.n_heads = n_heads; a.n_kv_heads = n_kv_heads; a.head_dim = head_dim;
  a.v_dim = v_dim; a.q_norm_w = q_norm_w; a.k_norm_w = k_norm_w; a.eps = eps;
  a.cos_table = cos_table; a.sin_table = sin_table; a.rotary_dim = cos_table ? rotary_dim : 0; a.table_rows = table_rows;
  a.interleaved = interleaved;
  a.token_seq = token_seq; a.token_pos = token_pos; a.seq_slot = seq_slot; a.seq_qstart = seq_qstart;
  a.page_table = page_table; a.table_stride = table_stride; a.num_pages = num_pages;
  a.k_pages = k_pages; a.v_pages = v_pages; a.write_cache = write_cache; a.status = status;
  x.temp_coef = temp_coef; x.temp_every = temp_every;
  auto al16 = [](const void* p) { return (uintptr_t)p % 16 == 0; };
  const long long all8 = ((long long)(n_heads + n_kv_heads) * head_dim + (long long)n_kv_heads * v_dim) / 8;
  const bool vec8 = dtype == PE_BF16 && a.rotary_dim == 0 && head_dim % 8 == 0 && v_dim % 8 == 0 && ld % 8 == 0 && al16(qkv) &&
                    al16(k_pages) && al16(v_pages) && al16(q_norm_w) && al16(k_norm_w) && all8 <= 4096;
  if (vec8) {
    // a few tokens (decode): one piece a thread, the shortest chain; many: two pieces a thread in flight
    int threads = (int)((n_tokens < 256 ? all8 : (all8 + 1) / 2) + 31) / 32 * 32;
    if (threads > 1024) threads = 1024;
    if (threads < 32) threads = 32;
    const int vpt = (int)((all8 + threads - 1) / threads);
    if (vpt <= 1) pe::launch(pe::qkv_row_norm_append_vec8_kernel<1>, n_tokens, threads, 0, stream, x);
    else if (vpt <= 2) pe::launch(pe::qkv_row_norm_append_vec8_kernel<2>, n_tokens, threads, 0, stream, x);
    else pe::launch(pe::qkv_row_norm_append_vec8_kernel<4>, n_tokens, threads, 0, stream, x);
  } else if (dtype == PE_F32) {
    pe::launch(pe::qkv_row_norm_append_kernel<float>, n_tokens, 256, 0, stream, x);
  } else {
    pe::launch(pe::qkv_row_norm_append_kernel<__nv_bfloat16>, n_tokens, 256, 0, stream, x);
  }
  PE_LAUNCH_CHECK();
  return PE_OK;
}
