// Several residual streams side by side, and layer norm.
//
// A block that keeps s copies X_1 .. X_s of the residual row (float32, [n, s, width]) reads a mix of them, and writes a
// sublayer's output y back into all of them at once:
//
//   write:   X_t <- sum_i mix[i, t] X_i + write[t] * (y + bias)       (every new stream from the old ones; mix is [from, to])
//   read:    u = sum_i read[i] X_i
//   norm:    layer norm (u - mean) / sqrt(mean((u - mean)^2) + eps) * w, or RMS norm u / sqrt(mean(u^2) + eps) * w
//
// One pass does the write of one sublayer, the read of the next and its norm: the streams go through memory once per
// sublayer.  Everything is float32; only y and the normed row have the run dtype.  With one stream and unit coefficients
// the same kernel is the usual residual add with a norm behind it.
//
// Modes: `single` given: the streams do not exist yet and are all equal to that row ([n, width]); the write makes them.
//        `y` null: nothing is written, only read.
//        `rows` given: output row r comes from stream row rows[r] and nothing is written back (the last norm).
#include "api.h"
#include "common.cuh"

namespace pe {

constexpr int kMaxStreams = 32;

struct StreamArgs {
  const float* single;   // [n, width] or null
  float* x;              // [n, s, width]
  const void* y;         // [n, width] run dtype, or null
  const float* bias;     // [width] or null
  const float* mix;      // [s, s]
  const float* write;    // [s]
  const float* read;     // [s]
  int norm;              // 0: none (out is float32), 1: layer norm, 2: RMS norm
  const float* w;        // [width]
  float eps;
  void* out;             // [n_rows, width]
  const int* rows;
  int n_rows, s, width;
};

template <typename T> __device__ __forceinline__ float4 stream_load4(const T* p);
template <> __device__ __forceinline__ float4 stream_load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 stream_load4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T> __device__ __forceinline__ void stream_store4(T* p, float4 v);
template <> __device__ __forceinline__ void stream_store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void stream_store4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<const uint32_t*>(&a);
  u.y = *reinterpret_cast<const uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}

// The norm of the row of `width` floats in `row` (every thread has filled its own places, stride blockDim * STEP), written
// to `out`; mean and mean square deviation are two sums, one after the other.
template <typename T, int STEP>
__device__ __forceinline__ void norm_row(const StreamArgs& a, const float* row, float sum, float* red, T* out) {
  const float n = (float)a.width;
  float mean = 0.f;
  float ss = 0.f;
  if (a.norm == 1) mean = block_sum(sum, red) / n;
  for (int c = threadIdx.x * STEP; c < a.width; c += blockDim.x * STEP)
#pragma unroll
    for (int e = 0; e < STEP; ++e) {
      const float d = row[c + e] - mean;
      ss = fmaf(d, d, ss);
    }
  const float inv = rsqrtf(block_sum(ss, red) / n + a.eps);
  for (int c = threadIdx.x * STEP; c < a.width; c += blockDim.x * STEP) {
    if (STEP == 4) {
      const float4 h = *reinterpret_cast<const float4*>(row + c), w = *reinterpret_cast<const float4*>(a.w + c);
      stream_store4<T>(out + c, make_float4((h.x - mean) * inv * w.x, (h.y - mean) * inv * w.y, (h.z - mean) * inv * w.z,
                                            (h.w - mean) * inv * w.w));
    } else {
      out[c] = from_f32<T>((row[c] - mean) * inv * a.w[c]);
    }
  }
}

// S streams known at compile time, 16-byte accesses (width a multiple of 4).  grid: rows; block: up to 1024 threads (512 from four streams on).
template <typename T, int S>
__global__ void __launch_bounds__(S >= 4 ? 512 : 1024) streams_vec4_kernel(StreamArgs a) {
  extern __shared__ __align__(16) float row_buf[];   // width floats
  __shared__ float red[32];
  // the coefficients do not come from the kernels before this one
  float mix[S][S], wr[S], rd[S];
#pragma unroll
  for (int i = 0; i < S; ++i) {
    rd[i] = a.read[i];
    wr[i] = a.y ? a.write[i] : 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) mix[i][t] = a.y ? a.mix[i * S + t] : 0.f;
  }
  // nor do the norm's weight and the bias: on their way to L2 (a decode step has streamed gigabytes of other weights through
  // it since the last one) while that kernel may still be running; one request a 128-byte line
  if (a.n_rows < kSMs && (threadIdx.x & 7) == 0)
    for (int c = threadIdx.x * 4; c < a.width; c += blockDim.x * 4) {
      if (a.w) asm volatile("prefetch.global.L2 [%0];\n" ::"l"(a.w + c));
      if (a.bias && a.y) asm volatile("prefetch.global.L2 [%0];\n" ::"l"(a.bias + c));
    }
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= a.n_rows) return;
  const size_t src = a.rows ? (size_t)a.rows[r] : (size_t)r;
  const int W = a.width;
  const float* single = a.single ? a.single + src * W : nullptr;
  float* x = a.x + src * S * W;
  const T* y = a.y ? (const T*)a.y + src * W : nullptr;
  const bool write_back = y != nullptr && a.rows == nullptr;
  float sum = 0.f;
  for (int c = threadIdx.x * 4; c < W; c += blockDim.x * 4) {
    float4 v[S];
    if (single) {
      const float4 one = *reinterpret_cast<const float4*>(single + c);
#pragma unroll
      for (int i = 0; i < S; ++i) v[i] = one;
    } else {
#pragma unroll
      for (int i = 0; i < S; ++i) v[i] = *reinterpret_cast<const float4*>(x + (size_t)i * W + c);
    }
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
    if (y) {
      float4 d = stream_load4<T>(y + c);
      if (a.bias) {
        const float4 b = *reinterpret_cast<const float4*>(a.bias + c);
        d.x += b.x; d.y += b.y; d.z += b.z; d.w += b.w;
      }
#pragma unroll
      for (int t = 0; t < S; ++t) {
        float4 n = make_float4(wr[t] * d.x, wr[t] * d.y, wr[t] * d.z, wr[t] * d.w);
#pragma unroll
        for (int i = 0; i < S; ++i) {
          n.x = fmaf(mix[i][t], v[i].x, n.x);
          n.y = fmaf(mix[i][t], v[i].y, n.y);
          n.z = fmaf(mix[i][t], v[i].z, n.z);
          n.w = fmaf(mix[i][t], v[i].w, n.w);
        }
        if (write_back) *reinterpret_cast<float4*>(x + (size_t)t * W + c) = n;
        u.x = fmaf(rd[t], n.x, u.x); u.y = fmaf(rd[t], n.y, u.y); u.z = fmaf(rd[t], n.z, u.z); u.w = fmaf(rd[t], n.w, u.w);
      }
    } else {
#pragma unroll
      for (int i = 0; i < S; ++i) {
        u.x = fmaf(rd[i], v[i].x, u.x); u.y = fmaf(rd[i], v[i].y, u.y); u.z = fmaf(rd[i], v[i].z, u.z); u.w = fmaf(rd[i], v[i].w, u.w);
      }
    }
    if (a.norm == 0) {
      *reinterpret_cast<float4*>((float*)a.out + (size_t)r * W + c) = u;
    } else {
      *reinterpret_cast<float4*>(row_buf + c) = u;
      sum += (u.x + u.y) + (u.z + u.w);
    }
  }
  if (a.norm != 0) norm_row<T, 4>(a, row_buf, sum, red, (T*)a.out + (size_t)r * W);
}

// Any number of streams up to kMaxStreams, any width.
template <typename T>
__global__ void streams_any_kernel(StreamArgs a) {
  extern __shared__ __align__(16) float smem[];      // width floats | mix | write | read
  __shared__ float red[32];
  const int W = a.width, S = a.s;
  float* row_buf = smem;
  float* mix = smem + W;
  float* wr = mix + S * S;
  float* rd = wr + S;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) mix[i] = a.y ? a.mix[i] : 0.f;
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    wr[i] = a.y ? a.write[i] : 0.f;
    rd[i] = a.read[i];
  }
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= a.n_rows) return;
  const size_t src = a.rows ? (size_t)a.rows[r] : (size_t)r;
  const float* single = a.single ? a.single + src * W : nullptr;
  float* x = a.x + src * S * W;
  const T* y = a.y ? (const T*)a.y + src * W : nullptr;
  const bool write_back = y != nullptr && a.rows == nullptr;
  float sum = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    float v[kMaxStreams];
    for (int i = 0; i < S; ++i) v[i] = single ? single[c] : x[(size_t)i * W + c];
    float u = 0.f;
    if (y) {
      const float d = to_f32<T>(y[c]) + (a.bias ? a.bias[c] : 0.f);
      for (int t = 0; t < S; ++t) {
        float n = wr[t] * d;
        for (int i = 0; i < S; ++i) n = fmaf(mix[i * S + t], v[i], n);
        if (write_back) x[(size_t)t * W + c] = n;
        u = fmaf(rd[t], n, u);
      }
    } else {
      for (int i = 0; i < S; ++i) u = fmaf(rd[i], v[i], u);
    }
    if (a.norm == 0) {
      ((float*)a.out)[(size_t)r * W + c] = u;
    } else {
      row_buf[c] = u;
      sum += u;
    }
  }
  if (a.norm != 0) norm_row<T, 1>(a, row_buf, sum, red, (T*)a.out + (size_t)r * W);
}

// Layer norm of rows in the run dtype.
template <typename T>
__global__ void layernorm_rows_kernel(const T* x, const float* __restrict__ w, T* __restrict__ out, int n_rows, int width, float eps) {
  extern __shared__ float row_buf[];
  __shared__ float red[32];
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  float sum = 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float h = to_f32<T>(x[(size_t)r * width + c]);
    row_buf[c] = h;
    sum += h;
  }
  const float mean = block_sum(sum, red) / (float)width;
  float ss = 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float d = row_buf[c] - mean;
    ss = fmaf(d, d, ss);
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)width + eps);
  for (int c = threadIdx.x; c < width; c += blockDim.x)
    out[(size_t)r * width + c] = from_f32<T>((row_buf[c] - mean) * inv * w[c]);
}

template <typename T>
static int launch_streams(const StreamArgs& a, cudaStream_t stream) {
  auto al = [](const void* p, size_t n) { return (uintptr_t)p % n == 0; };
  const size_t row_bytes = (size_t)a.width * sizeof(float);
  const bool vec = a.width % 4 == 0 && al(a.single, 16) && al(a.x, 16) && al(a.y, 4 * sizeof(T)) && al(a.bias, 16) && al(a.w, 16) &&
                   al(a.out, a.norm ? 4 * sizeof(T) : 16);
  auto go = [&](auto kern, int threads, size_t smem) -> int {
    if (smem > 200 * 1024) return PE_ERR_UNSUPPORTED_SIZE;
    if (smem > 48 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
    }
    pe::launch(kern, a.n_rows, threads, smem, stream, a);
    PE_LAUNCH_CHECK();
    return PE_OK;
  };
  if (vec && a.s <= 8) {
    // few rows (a decode step): as many threads as a row has pieces; many rows: smaller blocks, more of them on an SM
    const int pieces = (a.width / 4 + 31) / 32 * 32;
    const int most = a.n_rows >= 4 * kSMs ? 256 : (a.s >= 4 ? 512 : 1024);
    const int threads = pieces < most ? pieces : most;
    switch (a.s) {
      case 1: return go(streams_vec4_kernel<T, 1>, threads, row_bytes);
      case 2: return go(streams_vec4_kernel<T, 2>, threads, row_bytes);
      case 3: return go(streams_vec4_kernel<T, 3>, threads, row_bytes);
      case 4: return go(streams_vec4_kernel<T, 4>, threads, row_bytes);
      case 5: return go(streams_vec4_kernel<T, 5>, threads, row_bytes);
      case 6: return go(streams_vec4_kernel<T, 6>, threads, row_bytes);
      case 7: return go(streams_vec4_kernel<T, 7>, threads, row_bytes);
      default: return go(streams_vec4_kernel<T, 8>, threads, row_bytes);
    }
  }
  return go(streams_any_kernel<T>, 256, row_bytes + (size_t)(a.s * a.s + 2 * a.s) * sizeof(float));
}

}  // namespace pe

extern "C" int pe_stream_mix(int dtype, const float* single, float* x, const void* y, const float* bias, const float* mix,
                             const float* write, const float* read, int norm, const float* w, float eps, void* out, const int* rows,
                             int n_rows, int streams, int width, cudaStream_t stream) {
  if (n_rows <= 0) return PE_OK;
  if (streams <= 0 || streams > pe::kMaxStreams || width <= 0 || norm < 0 || norm > 2) return PE_ERR_UNSUPPORTED_SIZE;
  if (x == nullptr && (single == nullptr || y != nullptr)) return PE_ERR_BAD_ARGUMENT;
  if (read == nullptr || out == nullptr || (norm && w == nullptr) || (y && (mix == nullptr || write == nullptr))) return PE_ERR_BAD_ARGUMENT;
  pe::StreamArgs a;
  a.single = single; a.x = x; a.y = y; a.bias = bias; a.mix = mix; a.write = write; a.read = read; a.norm = norm; a.w = w;
  a.eps = eps; a.out = out; a.rows = rows; a.n_rows = n_rows; a.s = streams; a.width = width;
  if (dtype == PE_F32) return pe::launch_streams<float>(a, stream);
  if (dtype == PE_BF16) return pe::launch_streams<__nv_bfloat16>(a, stream);
  return PE_ERR_UNSUPPORTED_DTYPE;
}

extern "C" int pe_layernorm(int dtype, const void* x, const float* w, void* out, int n_rows, int width, float eps, cudaStream_t stream) {
  if (n_rows <= 0) return PE_OK;
  const size_t smem = (size_t)width * sizeof(float);
  if (width <= 0 || smem > 48 * 1024) return PE_ERR_UNSUPPORTED_SIZE;
  if (dtype == PE_F32)
    pe::launch(pe::layernorm_rows_kernel<float>, n_rows, 256, smem, stream, (const float*)x, w, (float*)out, n_rows, width, eps);
  else if (dtype == PE_BF16)
    pe::launch(pe::layernorm_rows_kernel<__nv_bfloat16>, n_rows, 256, smem, stream, (const __nv_bfloat16*)x, w, (__nv_bfloat16*)out,
               n_rows, width, eps);
  else
    return PE_ERR_UNSUPPORTED_DTYPE;
  PE_LAUNCH_CHECK();
  return PE_OK;
}
