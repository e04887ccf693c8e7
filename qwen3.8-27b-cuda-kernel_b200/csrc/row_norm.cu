// RMS-norm kernels of the layer-list architectures: embedding + first norm, post-norm + residual sum + next pre-norm,
// and the final norm of the rows the output head needs. One CTA per row; the row lives in shared memory between the
// passes, so global memory sees each operand once. Norms, the residual and its sum are fp32.
#include <algorithm>

#include "act.cuh"
#include "host_util.h"

namespace q38 {
Q38_REGISTER_ERROR_WORD();
namespace {

constexpr int kNormThreads = 256;

__device__ __forceinline__ float inv_rms(float sum_sq, int width, float eps) { return 1.0f / sqrtf(sum_sq / float(width) + eps); }

template <typename T>
__device__ __forceinline__ void store_normed(const float* row, int width, float rs, const q38_norm& norm, T* out, int ld) {
  for (int i = threadIdx.x; i < width; i += blockDim.x) out[i] = from_f32<T>(row[i] * rs * norm.gain[i * norm.gain_stride]);
}

template <typename T>
__global__ void __launch_bounds__(kNormThreads)
embed_norm_kernel(const __nv_bfloat16* __restrict__ table, const __nv_bfloat16* __restrict__ positions,
                  const int32_t* __restrict__ tokens, const int* __restrict__ tok_pos, int width,
                  float* __restrict__ residual, q38_norm norm, T* __restrict__ out, int ld) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ float row[];
  __shared__ float red[33];
  const int m = blockIdx.x;
  const __nv_bfloat16* e = table + (size_t)tokens[m] * width;
  const __nv_bfloat16* p = positions ? positions + (size_t)tok_pos[m] * width : nullptr;
  float ss = 0.0f;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    float x = __bfloat162float(e[i]);
    if (p) x += __bfloat162float(p[i]);
    residual[(size_t)m * width + i] = x;
    row[i] = x;
    ss += x * x;
  }
  const float rs = inv_rms(block_sum(ss, red), width, norm.eps);
  store_normed(row, width, rs, norm, out + (size_t)m * ld, ld);
}

template <typename T>
__global__ void __launch_bounds__(kNormThreads)
residual_norm_kernel(const float* __restrict__ y, int ldy, int width, q38_norm post, float* __restrict__ residual,
                     q38_norm next, T* __restrict__ out, int ld) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ float row[];
  __shared__ float red[33];
  const int m = blockIdx.x;
  const float* yr = y + (size_t)m * ldy;
  float* xr = residual + (size_t)m * width;
  float ss = 0.0f;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float v = yr[i];
    row[i] = v;
    ss += v * v;
  }
  const float rs = inv_rms(block_sum(ss, red), width, post.eps);
  ss = 0.0f;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float x = xr[i] + row[i] * (rs * post.gain[i * post.gain_stride]);
    xr[i] = x;
    row[i] = x;
    ss += x * x;
  }
  if (next.gain == nullptr) return;
  const float rs2 = inv_rms(block_sum(ss, red), width, next.eps);
  store_normed(row, width, rs2, next, out + (size_t)m * ld, ld);
}

__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
// The same with the row in registers, 16 elements per thread (rows in whole 16-byte pieces, up to 16384 elements): both
// operands are requested at once, and the two reductions are all that is left between them and the stores.
constexpr int kVecs = 4;
template <typename T>
__global__ void __launch_bounds__(1024)
residual_norm_vec_kernel(const float* __restrict__ y, int ldy, int width, q38_norm post, float* __restrict__ residual,
                         q38_norm next, T* __restrict__ out, int ld) {
  pdl_wait();
  pdl_launch_dependents();
  __shared__ float red[33];
  const int m = blockIdx.x;
  const float* yr = y + (size_t)m * ldy;
  float* xr = residual + (size_t)m * width;
  float4 v[kVecs], x[kVecs];
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < kVecs; ++i) {
    const int c = 4 * (threadIdx.x + i * blockDim.x);
    v[i] = x[i] = make_float4(0, 0, 0, 0);
    if (c < width) {
      v[i] = *reinterpret_cast<const float4*>(yr + c);
      x[i] = *reinterpret_cast<const float4*>(xr + c);
    }
  }
#pragma unroll
  for (int i = 0; i < kVecs; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
  const float rs = inv_rms(block_sum(ss, red), width, post.eps);
  ss = 0.0f;
  auto gains = [](const q38_norm& n, int c) {
    return n.gain_stride ? make_float4(n.gain[c], n.gain[c + 1], n.gain[c + 2], n.gain[c + 3])
                         : make_float4(n.gain[0], n.gain[0], n.gain[0], n.gain[0]);
  };
#pragma unroll
  for (int i = 0; i < kVecs; ++i) {
    const int c = 4 * (threadIdx.x + i * blockDim.x);
    if (c >= width) continue;
    const float4 g = gains(post, c);
    x[i].x += v[i].x * (rs * g.x);
    x[i].y += v[i].y * (rs * g.y);
    x[i].z += v[i].z * (rs * g.z);
    x[i].w += v[i].w * (rs * g.w);
    *reinterpret_cast<float4*>(xr + c) = x[i];
    ss += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
  }
  if (next.gain == nullptr) return;
  const float rs2 = inv_rms(block_sum(ss, red), width, next.eps);
#pragma unroll
  for (int i = 0; i < kVecs; ++i) {
    const int c = 4 * (threadIdx.x + i * blockDim.x);
    if (c >= width) continue;
    const float4 g = gains(next, c);
    store4(out + (size_t)m * ld + c, make_float4(x[i].x * rs2 * g.x, x[i].y * rs2 * g.y, x[i].z * rs2 * g.z, x[i].w * rs2 * g.w));
  }
}

template <typename T>
__global__ void __launch_bounds__(kNormThreads)
gather_norm_kernel(const float* __restrict__ residual, const int* __restrict__ rows, int first, int width, q38_norm norm,
                   T* __restrict__ out, int ld) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ float row[];
  __shared__ float red[33];
  const int src = rows ? rows[blockIdx.x] : first + int(blockIdx.x);
  const float* x = residual + (size_t)src * width;
  float ss = 0.0f;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float v = x[i];
    row[i] = v;
    ss += v * v;
  }
  const float rs = inv_rms(block_sum(ss, red), width, norm.eps);
  store_normed(row, width, rs, norm, out + (size_t)blockIdx.x * ld, ld);
}

int check_row(int m, int width, int ld, int act) {
  Q38_REQUIRE(m > 0 && width > 0 && width <= 12288 && ld >= width, "norm: rows %d, width %d, ld %d", m, width, ld);
  Q38_REQUIRE(act == Q38_ACT_BF16 || act == Q38_ACT_F32, "norm: activation precision %d", act);
  return Q38_OK;
}

}  // namespace
}  // namespace q38

using namespace q38;

extern "C" int q38_embed_norm(const q38_bf16* table, const q38_bf16* positions, const int32_t* tokens, const int* tok_pos,
                              int m, int width, float* residual, const q38_norm* norm, void* out, int ld_out, int act,
                              void* stream) {
  if (m == 0) return Q38_OK;
  Q38_REQUIRE(table && tokens && residual && norm && norm->gain && out && (tok_pos || !positions), "embed_norm: null argument");
  if (const int rc = check_row(m, width, ld_out, act)) return rc;
  const size_t smem = size_t(width) * 4;
  const auto* t = reinterpret_cast<const __nv_bfloat16*>(table);
  const auto* p = reinterpret_cast<const __nv_bfloat16*>(positions);
  if (act == Q38_ACT_BF16)
    (void)launch_kernel(embed_norm_kernel<__nv_bfloat16>, dim3(m), dim3(kNormThreads), smem, as_stream(stream), t, p, tokens,
                        tok_pos, width, residual, *norm, static_cast<__nv_bfloat16*>(out), ld_out);
  else
    (void)launch_kernel(embed_norm_kernel<float>, dim3(m), dim3(kNormThreads), smem, as_stream(stream), t, p, tokens, tok_pos,
                        width, residual, *norm, static_cast<float*>(out), ld_out);
  Q38_LAUNCH_OK("embed_norm_kernel");
  return Q38_OK;
}

extern "C" int q38_residual_norm(const float* y, int ldy, int m, int width, const q38_norm* post, float* residual,
                                 const q38_norm* next, void* out, int ld_out, int act, void* stream) {
  if (m == 0) return Q38_OK;
  Q38_REQUIRE(y && post && post->gain && residual && (!next || (next->gain && out)), "residual_norm: null argument");
  if (const int rc = check_row(m, width, next ? ld_out : width, act)) return rc;
  Q38_REQUIRE(ldy >= width, "residual_norm: ldy %d", ldy);
  const size_t smem = size_t(width) * 4;
  const q38_norm nx = next ? *next : q38_norm{nullptr, 0, 0.0f};
  if (width % 4 == 0 && ldy % 4 == 0 && (!next || ld_out % 4 == 0) && width <= 16384 &&
      (reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(residual) | reinterpret_cast<uintptr_t>(out)) % 16 == 0) {
    const int threads = std::max(64, std::min(1024, (width / (4 * kVecs) + 31) / 32 * 32));
    if (act == Q38_ACT_BF16)
      (void)launch_kernel(residual_norm_vec_kernel<__nv_bfloat16>, dim3(m), dim3(threads), 0, as_stream(stream), y, ldy, width, *post,
                          residual, nx, static_cast<__nv_bfloat16*>(out), ld_out);
    else
      (void)launch_kernel(residual_norm_vec_kernel<float>, dim3(m), dim3(threads), 0, as_stream(stream), y, ldy, width, *post, residual,
                          nx, static_cast<float*>(out), ld_out);
    Q38_LAUNCH_OK("residual_norm_vec_kernel");
    return Q38_OK;
  }
  if (act == Q38_ACT_BF16)
    (void)launch_kernel(residual_norm_kernel<__nv_bfloat16>, dim3(m), dim3(kNormThreads), smem, as_stream(stream), y, ldy, width,
                        *post, residual, nx, static_cast<__nv_bfloat16*>(out), ld_out);
  else
    (void)launch_kernel(residual_norm_kernel<float>, dim3(m), dim3(kNormThreads), smem, as_stream(stream), y, ldy, width, *post,
                        residual, nx, static_cast<float*>(out), ld_out);
  Q38_LAUNCH_OK("residual_norm_kernel");
  return Q38_OK;
}

extern "C" int q38_gather_norm(const float* residual, const int* rows, int first, int n, int width, const q38_norm* norm,
                               void* out, int ld_out, int act, void* stream) {
  if (n == 0) return Q38_OK;
  Q38_REQUIRE(residual && norm && norm->gain && out && first >= 0, "gather_norm: arguments");
  if (const int rc = check_row(n, width, ld_out, act)) return rc;
  const size_t smem = size_t(width) * 4;
  if (act == Q38_ACT_BF16)
    (void)launch_kernel(gather_norm_kernel<__nv_bfloat16>, dim3(n), dim3(kNormThreads), smem, as_stream(stream), residual, rows,
                        first, width, *norm, static_cast<__nv_bfloat16*>(out), ld_out);
  else
    (void)launch_kernel(gather_norm_kernel<float>, dim3(n), dim3(kNormThreads), smem, as_stream(stream), residual, rows, first,
                        width, *norm, static_cast<float*>(out), ld_out);
  Q38_LAUNCH_OK("gather_norm_kernel");
  return Q38_OK;
}
