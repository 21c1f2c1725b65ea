// RMSNorm over the last dimension with the residual add fused in.
//
//   h   = residual[row] (+ delta[row])            float32
//   out = h * rsqrt(mean(h^2) + eps) * w          float32 math, stored in the run dtype
//
// Reference formulas: pygguf_engine/quant_kernels.py:1595-1596 (add, then norm), 831-833 (mean,
// rsqrt, multiply in float32), weight held in float32 (pygguf_engine/model.py:63).
// Modes:  rows == nullptr: row r of the output is row r of the stream; with `delta` the sum is
//         written back to the stream (the residual add of the block).
//         rows != nullptr: output row r is stream row rows[r] (+ delta row rows[r]); nothing is
//         written back (the final norm on the rows whose logits are wanted).
#include "api.h"
#include "common.cuh"

namespace pe {

template <typename TDelta, typename TOut>
__global__ void rmsnorm_kernel(float* __restrict__ residual, const TDelta* delta,
                               const float* __restrict__ weight, TOut* __restrict__ out,
                               const int* rows, int n_rows, int dim, float eps) {
  extern __shared__ float row_buf[];  // dim floats
  __shared__ float red[32];
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  float* res_row = residual + src * dim;
  const TDelta* d_row = delta ? delta + src * dim : nullptr;
  float ss = 0.f;
  for (int c = threadIdx.x; c < dim; c += blockDim.x) {
    float h = res_row[c];
    if (d_row) h += to_f32<TDelta>(d_row[c]);
    row_buf[c] = h;
    ss += h * h;
  }
  const float total = block_sum(ss, red);
  const float inv = rsqrtf(total / (float)dim + eps);
  const bool write_back = (d_row != nullptr) && (rows == nullptr);
  TOut* o_row = out + (size_t)r * dim;
  for (int c = threadIdx.x; c < dim; c += blockDim.x) {
    const float h = row_buf[c];
    if (write_back) res_row[c] = h;
    o_row[c] = from_f32<TOut>(h * inv * weight[c]);
  }
}

// The same with 4-element accesses (16-byte loads and stores of the float32 stream), for widths that
// are a multiple of 4; rows then start on 16-byte boundaries.
template <typename T> struct Vec4;
template <> struct Vec4<float> {
  static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Vec4<__nv_bfloat16> {
  static __device__ __forceinline__ float4 load(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&u.x), b = *reinterpret_cast<const __nv_bfloat162*>(&u.y);
    return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<uint32_t*>(&a);
    u.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
  }
};

template <typename TDelta, typename TOut>
__global__ void __launch_bounds__(1024) rmsnorm_vec4_kernel(float* __restrict__ residual, const TDelta* delta,
                                                             const float* __restrict__ weight, TOut* __restrict__ out,
                                                             const int* rows, int n_rows, int dim, float eps) {
  extern __shared__ float row_buf[];  // dim floats
  __shared__ float red[32];
  // The norm's weight does not depend on the kernels before this one: the part of it that this thread
  // needs first is on its way before the wait (a decode step waits for this kernel's latency 73 times).
  const int c0 = threadIdx.x * 4;
  float4 w0 = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c0 < dim) w0 = Vec4<float>::load(weight + c0);
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  float* res_row = residual + src * dim;
  const TDelta* d_row = delta ? delta + src * dim : nullptr;
  const bool write_back = (d_row != nullptr) && (rows == nullptr);
  float ss = 0.f;
  for (int c = c0; c < dim; c += blockDim.x * 4) {
    float4 h = Vec4<float>::load(res_row + c);
    if (d_row) {
      const float4 d = Vec4<TDelta>::load(d_row + c);
      h.x += d.x; h.y += d.y; h.z += d.z; h.w += d.w;
      if (write_back) Vec4<float>::store(res_row + c, h);
    }
    *reinterpret_cast<float4*>(row_buf + c) = h;
    ss += h.x * h.x + h.y * h.y + h.z * h.z + h.w * h.w;
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)dim + eps);
  TOut* o_row = out + (size_t)r * dim;
  for (int c = c0; c < dim; c += blockDim.x * 4) {
    const float4 h = *reinterpret_cast<const float4*>(row_buf + c);
    const float4 w = c == c0 ? w0 : Vec4<float>::load(weight + c);
    Vec4<TOut>::store(o_row + c, make_float4(h.x * inv * w.x, h.y * inv * w.y, h.z * inv * w.z, h.w * inv * w.w));
  }
}

// Plain RMSNorm of a tensor in the run dtype (rows of any width), used by parts that normalise
// something other than the residual stream.
template <typename T>
__global__ void rmsnorm_plain_kernel(const T* x, long long x_ld, const float* __restrict__ weight, T* __restrict__ out,
                                     int n_rows, int dim, float eps) {
  extern __shared__ float row_buf[];
  __shared__ float red[32];
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  float ss = 0.f;
  for (int c = threadIdx.x; c < dim; c += blockDim.x) {
    const float h = to_f32<T>(x[(size_t)r * x_ld + c]);
    row_buf[c] = h;
    ss += h * h;
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)dim + eps);
  for (int c = threadIdx.x; c < dim; c += blockDim.x)
    out[(size_t)r * dim + c] = from_f32<T>(row_buf[c] * inv * weight[c]);
}

// The same for rows in 4-element pieces that a block holds in registers (up to VPT pieces a thread).
template <typename T, int VPT>
__global__ void __launch_bounds__(1024) rmsnorm_plain_vec4_kernel(const T* x, long long x_ld, const float* __restrict__ weight,
                                                                   T* __restrict__ out, int dim, float eps) {
  __shared__ float red[32];
  pdl_wait_block();
  pdl_launch_dependents();
  const T* row = x + (size_t)blockIdx.x * x_ld;
  float4 h[VPT];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 4;
    h[k] = c < dim ? Vec4<T>::load(row + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) ss += h[k].x * h[k].x + h[k].y * h[k].y + h[k].z * h[k].z + h[k].w * h[k].w;
  const float inv = rsqrtf(block_sum(ss, red) / (float)dim + eps);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 4;
    if (c >= dim) break;
    const float4 w = Vec4<float>::load(weight + c);
    Vec4<T>::store(out + (size_t)blockIdx.x * dim + c, make_float4(h[k].x * inv * w.x, h[k].y * inv * w.y, h[k].z * inv * w.z, h[k].w * inv * w.w));
  }
}

// Norm on a sublayer's output, then the residual add (a block that norms what it adds, not what it reads):
//   stream[row] += delta[row] * rsqrt(mean(delta[row]^2) + eps) * w        float32
// and, when `cast` is given, cast[row] = stream[row] in the run dtype: the next sublayer's input.
template <typename T>
__global__ void rmsnorm_add_kernel(float* __restrict__ stream, const T* delta, const float* __restrict__ weight,
                                   T* __restrict__ cast, int n_rows, int dim, float eps) {
  extern __shared__ float row_buf[];  // dim floats
  __shared__ float red[32];
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  const T* d_row = delta + (size_t)r * dim;
  float ss = 0.f;
  for (int c = threadIdx.x; c < dim; c += blockDim.x) {
    const float y = to_f32<T>(d_row[c]);
    row_buf[c] = y;
    ss += y * y;
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)dim + eps);
  float* s_row = stream + (size_t)r * dim;
  for (int c = threadIdx.x; c < dim; c += blockDim.x) {
    const float h = s_row[c] + row_buf[c] * inv * weight[c];
    s_row[c] = h;
    if (cast) cast[(size_t)r * dim + c] = from_f32<T>(h);
  }
}

// The same with 4-element accesses, for widths that are a multiple of 4 and 16-byte aligned rows.
template <typename T>
__global__ void __launch_bounds__(1024) rmsnorm_add_vec4_kernel(float* __restrict__ stream, const T* delta,
                                                                 const float* __restrict__ weight, T* __restrict__ cast,
                                                                 int n_rows, int dim, float eps) {
  extern __shared__ float row_buf[];  // dim floats
  __shared__ float red[32];
  const int c0 = threadIdx.x * 4;
  float4 w0 = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c0 < dim) w0 = Vec4<float>::load(weight + c0);       // the weight does not come from the kernel before this one
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  const T* d_row = delta + (size_t)r * dim;
  float* s_row = stream + (size_t)r * dim;
  float ss = 0.f;
  float4 s0 = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c0 < dim) s0 = Vec4<float>::load(s_row + c0);        // the stream's first piece is on its way during the reduction
  for (int c = c0; c < dim; c += blockDim.x * 4) {
    const float4 y = Vec4<T>::load(d_row + c);
    *reinterpret_cast<float4*>(row_buf + c) = y;
    ss += y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w;
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)dim + eps);
  for (int c = c0; c < dim; c += blockDim.x * 4) {
    const float4 y = *reinterpret_cast<const float4*>(row_buf + c);
    const float4 w = c == c0 ? w0 : Vec4<float>::load(weight + c);
    float4 h = c == c0 ? s0 : Vec4<float>::load(s_row + c);
    h.x += y.x * inv * w.x; h.y += y.y * inv * w.y; h.z += y.z * inv * w.z; h.w += y.w * inv * w.w;
    Vec4<float>::store(s_row + c, h);
    if (cast) Vec4<T>::store(cast + (size_t)r * dim + c, h);
  }
}

// The add of several scaled sublayer outputs at once, then the norm (a block whose sublayers all read one norm's
// output and are added together):  h = residual[row] + sum_i scale_i * delta_i[row];  out = h * rsqrt(mean(h^2) + eps) * w.
// Modes as above: without `rows` the sum is written back to the stream, with `rows` nothing is.
struct DeltaList {
  const void* ptr[4];
  float scale[4];
  int count;
};

template <typename TDelta, typename TOut>
__global__ void rmsnorm_sum_kernel(float* __restrict__ residual, DeltaList deltas, const float* __restrict__ weight,
                                   TOut* __restrict__ out, const int* rows, int n_rows, int dim, float eps) {
  extern __shared__ float row_buf[];  // dim floats
  __shared__ float red[32];
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  float* res_row = residual + src * dim;
  float ss = 0.f;
  for (int c = threadIdx.x; c < dim; c += blockDim.x) {
    float h = res_row[c];
    for (int i = 0; i < deltas.count; ++i)
      h = fmaf(deltas.scale[i], to_f32<TDelta>(((const TDelta*)deltas.ptr[i])[src * dim + c]), h);
    row_buf[c] = h;
    ss += h * h;
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)dim + eps);
  const bool write_back = rows == nullptr;
  for (int c = threadIdx.x; c < dim; c += blockDim.x) {
    const float h = row_buf[c];
    if (write_back) res_row[c] = h;
    if (out) out[(size_t)r * dim + c] = from_f32<TOut>(h * inv * weight[c]);
  }
}

// The same with 4-element accesses, for widths that are a multiple of 4 and rows on 16-byte boundaries.
template <typename TDelta, typename TOut>
__global__ void __launch_bounds__(1024) rmsnorm_sum_vec4_kernel(float* __restrict__ residual, DeltaList deltas,
                                                                 const float* __restrict__ weight, TOut* __restrict__ out,
                                                                 const int* rows, int n_rows, int dim, float eps) {
  extern __shared__ float row_buf[];  // dim floats
  __shared__ float red[32];
  const int c0 = threadIdx.x * 4;
  float4 w0 = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c0 < dim) w0 = Vec4<float>::load(weight + c0);       // the weight does not come from the kernel before this one
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  float* res_row = residual + src * dim;
  const bool write_back = rows == nullptr;
  float ss = 0.f;
  for (int c = c0; c < dim; c += blockDim.x * 4) {
    float4 h = Vec4<float>::load(res_row + c);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      if (i < deltas.count) {
        const float4 d = Vec4<TDelta>::load((const TDelta*)deltas.ptr[i] + src * dim + c);
        const float sc = deltas.scale[i];
        h.x = fmaf(sc, d.x, h.x); h.y = fmaf(sc, d.y, h.y); h.z = fmaf(sc, d.z, h.z); h.w = fmaf(sc, d.w, h.w);
      }
    }
    if (write_back) Vec4<float>::store(res_row + c, h);
    *reinterpret_cast<float4*>(row_buf + c) = h;
    ss += h.x * h.x + h.y * h.y + h.z * h.z + h.w * h.w;
  }
  if (!out) return;
  const float inv = rsqrtf(block_sum(ss, red) / (float)dim + eps);
  TOut* o_row = out + (size_t)r * dim;
  for (int c = c0; c < dim; c += blockDim.x * 4) {
    const float4 h = *reinterpret_cast<const float4*>(row_buf + c);
    const float4 w = c == c0 ? w0 : Vec4<float>::load(weight + c);
    Vec4<TOut>::store(o_row + c, make_float4(h.x * inv * w.x, h.y * inv * w.y, h.z * inv * w.z, h.w * inv * w.w));
  }
}

// Norm behind the sum (the stream itself is what the norm returns):
//   h = alpha * stream[row] + scale * delta[row] ;  stream[row] = h * rsqrt(mean(h^2) + eps) * w          float32
// with one factor `scale` per feature (null: 1), and, when `cast` is given, cast[row] = stream[row] in the run dtype: the
// next sublayer's input.
template <typename T>
__global__ void rmsnorm_of_sum_kernel(float* __restrict__ stream, const T* delta, float alpha, const float* __restrict__ scale,
                                      const float* __restrict__ weight, T* __restrict__ cast, int n_rows, int dim, float eps) {
  extern __shared__ float row_buf[];  // dim floats
  __shared__ float red[32];
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  float* s_row = stream + (size_t)r * dim;
  const T* d_row = delta + (size_t)r * dim;
  float ss = 0.f;
  for (int c = threadIdx.x; c < dim; c += blockDim.x) {
    const float y = to_f32<T>(d_row[c]) * (scale ? scale[c] : 1.f);
    const float h = fmaf(alpha, s_row[c], y);
    row_buf[c] = h;
    ss += h * h;
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)dim + eps);
  for (int c = threadIdx.x; c < dim; c += blockDim.x) {
    const float h = row_buf[c] * inv * weight[c];
    s_row[c] = h;
    if (cast) cast[(size_t)r * dim + c] = from_f32<T>(h);
  }
}

// The same with 4-element accesses, for widths that are a multiple of 4 and 16-byte aligned rows; a thread keeps up to VPT
// pieces of the row in registers.
template <typename T, int VPT>
__global__ void __launch_bounds__(1024) rmsnorm_of_sum_vec4_kernel(float* __restrict__ stream, const T* delta, float alpha,
                                                                    const float* __restrict__ scale,
                                                                    const float* __restrict__ weight, T* __restrict__ cast,
                                                                    int n_rows, int dim, float eps) {
  __shared__ float red[32];
  const int c0 = threadIdx.x * 4, step = blockDim.x * 4;
  // neither the weight nor the factors come from the kernel before this one
  float4 f[VPT];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    f[k] = make_float4(1.f, 1.f, 1.f, 1.f);
    if (scale && c0 + k * step < dim) f[k] = Vec4<float>::load(scale + c0 + k * step);
  }
  float4 w0 = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c0 < dim) w0 = Vec4<float>::load(weight + c0);
  pdl_wait_block();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  float* s_row = stream + (size_t)r * dim;
  const T* d_row = delta + (size_t)r * dim;
  float4 h[VPT];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int c = c0 + k * step;
    h[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < dim) {
      const float4 x = Vec4<float>::load(s_row + c), y = Vec4<T>::load(d_row + c);
      h[k] = make_float4(fmaf(alpha, x.x, f[k].x * y.x), fmaf(alpha, x.y, f[k].y * y.y), fmaf(alpha, x.z, f[k].z * y.z),
                         fmaf(alpha, x.w, f[k].w * y.w));
    }
  }
#pragma unroll
  for (int k = 0; k < VPT; ++k) ss += h[k].x * h[k].x + h[k].y * h[k].y + h[k].z * h[k].z + h[k].w * h[k].w;
  const float inv = rsqrtf(block_sum(ss, red) / (float)dim + eps);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int c = c0 + k * step;
    if (c >= dim) break;
    const float4 w = k == 0 ? w0 : Vec4<float>::load(weight + c);
    const float4 o = make_float4(h[k].x * inv * w.x, h[k].y * inv * w.y, h[k].z * inv * w.z, h[k].w * inv * w.w);
    Vec4<float>::store(s_row + c, o);
    if (cast) Vec4<T>::store(cast + (size_t)r * dim + c, o);
  }
}

template <typename K>
static int set_smem(K kernel, size_t bytes) {
  if (bytes > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (e != cudaSuccess) return (int)e;
  }
  return 0;
}

}  // namespace pe

extern "C" int pe_rmsnorm_residual(int dtype, float* residual, const void* delta, const float* weight, void* out,
                                   const int* rows, int n_rows, int dim, float eps, cudaStream_t stream) {
  if (n_rows <= 0) return PE_OK;
  if (dim <= 0) return PE_ERR_BAD_ARGUMENT;
  const size_t smem = (size_t)dim * sizeof(float);
  if (smem > 200 * 1024) return PE_ERR_UNSUPPORTED_SIZE;  // rows wider than 51,200 features
  int threads = dim >= 2048 ? 512 : (dim >= 512 ? 256 : 128);
  int e;
  const bool vec = (dim % 4 == 0) && ((uintptr_t)residual % 16 == 0) && ((uintptr_t)weight % 16 == 0) &&
                   ((uintptr_t)out % 16 == 0) && ((uintptr_t)delta % 16 == 0);
  // A handful of rows (a decode step): what counts is the kernel's latency, and a thread that has a
  // second 16-byte piece to fetch waits for memory a second time (8B shape, batch 8: 3.97 ms a step with
  // 512 threads a row, 3.95 with 1,024, 4.08 with 256, 5.18 with 128).
  if (vec && n_rows <= 64 && dim > 2048) threads = 1024;
  if (dtype == PE_F32) {
    auto k = vec ? pe::rmsnorm_vec4_kernel<float, float> : pe::rmsnorm_kernel<float, float>;
    if ((e = pe::set_smem(k, smem))) return e;
    pe::launch(k, n_rows, threads, smem, stream, residual, (const float*)delta, weight, (float*)out, rows, n_rows, dim, eps);
  } else if (dtype == PE_BF16) {
    auto k = vec ? pe::rmsnorm_vec4_kernel<__nv_bfloat16, __nv_bfloat16> : pe::rmsnorm_kernel<__nv_bfloat16, __nv_bfloat16>;
    if ((e = pe::set_smem(k, smem))) return e;
    pe::launch(k, n_rows, threads, smem, stream, residual, (const __nv_bfloat16*)delta, weight, (__nv_bfloat16*)out, rows, n_rows, dim, eps);
  } else {
    return PE_ERR_UNSUPPORTED_DTYPE;
  }
  PE_LAUNCH_CHECK();
  return PE_OK;
}

// Rows of x lie x_ld elements apart; rows of out are packed.
extern "C" int pe_rmsnorm_rows(int dtype, const void* x, long long x_ld, const float* weight, void* out, int n_rows, int dim,
                               float eps, cudaStream_t stream) {
  if (n_rows <= 0) return PE_OK;
  if (dim <= 0 || x_ld < dim) return PE_ERR_BAD_ARGUMENT;
  if (dtype != PE_F32 && dtype != PE_BF16) return PE_ERR_UNSUPPORTED_DTYPE;
  const size_t smem = (size_t)dim * sizeof(float);
  if (smem > 200 * 1024) return PE_ERR_UNSUPPORTED_SIZE;
  const bool vec = dim % 4 == 0 && x_ld % 4 == 0 && dim <= 16384 && ((uintptr_t)x % 16 == 0) && ((uintptr_t)weight % 16 == 0) &&
                   ((uintptr_t)out % 16 == 0);
  if (vec) {
    int threads = (dim / 4 + 31) / 32 * 32;
    if (n_rows > 2 * pe::kSMs && threads > 256) threads = 256;
    if (threads > 1024) threads = 1024;
    while (threads < 1024 && dim > threads * 16) threads *= 2;
    const int vpt = (dim + threads * 4 - 1) / (threads * 4);
#define PE_ROWS(T, V) pe::launch(pe::rmsnorm_plain_vec4_kernel<T, V>, n_rows, threads, 0, stream, (const T*)x, x_ld, weight, (T*)out, dim, eps)
#define PE_ROWS_T(T)               \
  do {                             \
    if (vpt <= 1) PE_ROWS(T, 1);   \
    else if (vpt <= 2) PE_ROWS(T, 2); \
    else PE_ROWS(T, 4);            \
  } while (0)
    if (dtype == PE_F32) PE_ROWS_T(float);
    else PE_ROWS_T(__nv_bfloat16);
#undef PE_ROWS_T
#undef PE_ROWS
    PE_LAUNCH_CHECK();
    return PE_OK;
  }
  const int threads = dim >= 2048 ? 512 : (dim >= 512 ? 256 : 128);
  int e;
  if (dtype == PE_F32) {
    auto k = pe::rmsnorm_plain_kernel<float>;
    if ((e = pe::set_smem(k, smem))) return e;
    pe::launch(k, n_rows, threads, smem, stream, (const float*)x, x_ld, weight, (float*)out, n_rows, dim, eps);
  } else {
    auto k = pe::rmsnorm_plain_kernel<__nv_bfloat16>;
    if ((e = pe::set_smem(k, smem))) return e;
    pe::launch(k, n_rows, threads, smem, stream, (const __nv_bfloat16*)x, x_ld, weight, (__nv_bfloat16*)out, n_rows, dim, eps);
  }
  PE_LAUNCH_CHECK();
  return PE_OK;
}

extern "C" int pe_rmsnorm(int dtype, const void* x, const float* weight, void* out, int n_rows, int dim, float eps,
                          cudaStream_t stream) {
  return pe_rmsnorm_rows(dtype, x, dim, weight, out, n_rows, dim, eps, stream);
}

extern "C" int pe_rmsnorm_add(int dtype, float* stream, const void* delta, const float* weight, void* cast, int n_rows,
                              int dim, float eps, cudaStream_t stream_) {
  if (n_rows <= 0) return PE_OK;
  if (dim <= 0) return PE_ERR_BAD_ARGUMENT;
  const size_t smem = (size_t)dim * sizeof(float);
  if (smem > 200 * 1024) return PE_ERR_UNSUPPORTED_SIZE;
  int threads = dim >= 2048 ? 512 : (dim >= 512 ? 256 : 128);
  const bool vec = (dim % 4 == 0) && ((uintptr_t)stream % 16 == 0) && ((uintptr_t)weight % 16 == 0) &&
                   ((uintptr_t)cast % 16 == 0) && ((uintptr_t)delta % 16 == 0);
  if (vec && n_rows <= 64 && dim > 2048) threads = 1024;   // a handful of rows: latency counts (see pe_rmsnorm_residual)
  int e;
  if (dtype == PE_F32) {
    auto k = vec ? pe::rmsnorm_add_vec4_kernel<float> : pe::rmsnorm_add_kernel<float>;
    if ((e = pe::set_smem(k, smem))) return e;
    pe::launch(k, n_rows, threads, smem, stream_, stream, (const float*)delta, weight, (float*)cast, n_rows, dim, eps);
  } else if (dtype == PE_BF16) {
    auto k = vec ? pe::rmsnorm_add_vec4_kernel<__nv_bfloat16> : pe::rmsnorm_add_kernel<__nv_bfloat16>;
    if ((e = pe::set_smem(k, smem))) return e;
    pe::launch(k, n_rows, threads, smem, stream_, stream, (const __nv_bfloat16*)delta, weight, (__nv_bfloat16*)cast, n_rows, dim, eps);
  } else {
    return PE_ERR_UNSUPPORTED_DTYPE;
  }
  PE_LAUNCH_CHECK();
  return PE_OK;
}

extern "C" int pe_rmsnorm_residual_sum(int dtype, float* residual, const void* const* deltas, const float* scales, int n_deltas,
                                       const float* weight, void* out, const int* rows, int n_rows, int dim, float eps,
                                       cudaStream_t stream) {
  if (n_rows <= 0) return PE_OK;
  if (dim <= 0 || n_deltas < 0 || n_deltas > 4) return PE_ERR_BAD_ARGUMENT;
  const size_t smem = (size_t)dim * sizeof(float);
  if (smem > 200 * 1024) return PE_ERR_UNSUPPORTED_SIZE;
  pe::DeltaList list;
  list.count = n_deltas;
  for (int i = 0; i < 4; ++i) {
    list.ptr[i] = i < n_deltas ? deltas[i] : nullptr;
    list.scale[i] = i < n_deltas ? scales[i] : 0.f;
  }
  int threads = dim >= 2048 ? 512 : (dim >= 512 ? 256 : 128);
  bool vec = (dim % 4 == 0) && ((uintptr_t)residual % 16 == 0) && ((uintptr_t)weight % 16 == 0) && ((uintptr_t)out % 16 == 0);
  for (int i = 0; i < n_deltas; ++i) vec = vec && ((uintptr_t)deltas[i] % 16 == 0);
  if (vec && n_rows <= 64 && dim > 2048) threads = 1024;   // a handful of rows: latency counts (see pe_rmsnorm_residual)
  int e;
  if (dtype == PE_F32) {
    auto k = vec ? pe::rmsnorm_sum_vec4_kernel<float, float> : pe::rmsnorm_sum_kernel<float, float>;
    if ((e = pe::set_smem(k, smem))) return e;
    pe::launch(k, n_rows, threads, smem, stream, residual, list, weight, (float*)out, rows, n_rows, dim, eps);
  } else if (dtype == PE_BF16) {
    auto k = vec ? pe::rmsnorm_sum_vec4_kernel<__nv_bfloat16, __nv_bfloat16> : pe::rmsnorm_sum_kernel<__nv_bfloat16, __nv_bfloat16>;
    if ((e = pe::set_smem(k, smem))) return e;
    pe::launch(k, n_rows, threads, smem, stream, residual, list, weight, (__nv_bfloat16*)out, rows, n_rows, dim, eps);
  } else {
    return PE_ERR_UNSUPPORTED_DTYPE;
  }
  PE_LAUNCH_CHECK();
  return PE_OK;
}

extern "C" int pe_rmsnorm_of_sum(int dtype, float* stream, const void* delta, float alpha, const float* scale, const float* weight,
                                 void* cast, int n_rows, int dim, float eps, cudaStream_t stream_) {
  if (n_rows <= 0) return PE_OK;
  if (dim <= 0 || !stream || !delta || !weight) return PE_ERR_BAD_ARGUMENT;
  if (dtype != PE_F32 && dtype != PE_BF16) return PE_ERR_UNSUPPORTED_DTYPE;
  const size_t smem = (size_t)dim * sizeof(float);
  if (smem > 200 * 1024) return PE_ERR_UNSUPPORTED_SIZE;
  int threads = dim >= 2048 ? 512 : (dim >= 512 ? 256 : 128);
  const bool vec = (dim % 4 == 0) && dim <= 16384 && ((uintptr_t)stream % 16 == 0) && ((uintptr_t)weight % 16 == 0) &&
                   ((uintptr_t)scale % 16 == 0) && ((uintptr_t)cast % 16 == 0) && ((uintptr_t)delta % 16 == 0);
  if (vec && n_rows <= 64 && dim > 2048) threads = 1024;   // a handful of rows: latency counts (see pe_rmsnorm_residual)
  if (vec) {
    while (threads < 1024 && dim > threads * 16) threads *= 2;
    const int vpt = (dim + threads * 4 - 1) / (threads * 4);
#define PE_OF_SUM(T, V)                                                                                                        \
  pe::launch(pe::rmsnorm_of_sum_vec4_kernel<T, V>, n_rows, threads, 0, stream_, stream, (const T*)delta, alpha, scale, weight, \
             (T*)cast, n_rows, dim, eps)
#define PE_OF_SUM_T(T)               \
  do {                               \
    if (vpt <= 1) PE_OF_SUM(T, 1);   \
    else if (vpt <= 2) PE_OF_SUM(T, 2); \
    else PE_OF_SUM(T, 4);            \
  } while (0)
    if (dtype == PE_F32) PE_OF_SUM_T(float);
    else PE_OF_SUM_T(__nv_bfloat16);
#undef PE_OF_SUM_T
#undef PE_OF_SUM
  } else if (dtype == PE_F32) {
    int e;
    if ((e = pe::set_smem(pe::rmsnorm_of_sum_kernel<float>, smem))) return e;
    pe::launch(pe::rmsnorm_of_sum_kernel<float>, n_rows, threads, smem, stream_, stream, (const float*)delta, alpha, scale, weight,
               (float*)cast, n_rows, dim, eps);
  } else {
    int e;
    if ((e = pe::set_smem(pe::rmsnorm_of_sum_kernel<__nv_bfloat16>, smem))) return e;
    pe::launch(pe::rmsnorm_of_sum_kernel<__nv_bfloat16>, n_rows, threads, smem, stream_, stream, (const __nv_bfloat16*)delta, alpha,
               scale, weight, (__nv_bfloat16*)cast, n_rows, dim, eps);
  }
  PE_LAUNCH_CHECK();
  return PE_OK;
}
