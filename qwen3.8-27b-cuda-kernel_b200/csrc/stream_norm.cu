// Residual streams (hyper-connections) of the layer-list architectures: the streams' update after a sublayer, the next
// sublayer's weighted sum of them and its pre-norm in one pass over the row; the embedding in front and the sum of the
// streams at the end. Everything is fp32 up to the stored pre-norm. RMS norms over equal parts of the row (1 = all of it).
//
// One CTA per token. The new streams stay in registers only as long as they are written; u is kept in shared memory for
// the norm. With few tokens in the step the CTAs are wide, so that a row is one or two rounds of 16-byte pieces.
#include <algorithm>

#include "act.cuh"
#include "host_util.h"

namespace q38 {
Q38_REGISTER_ERROR_WORD();
namespace {

constexpr int kMaxThreads = 1024;

// What a row of u becomes: out = u / rms(part of u) * gain. `u` lives in shared memory, ssq holds a partial sum of squares
// per (part, slice) pair and then the parts' inverse root mean squares.
struct RowNorm {
  q38_norm n;
  int groups, part;  // equal parts of `part` elements
};

__device__ __forceinline__ void part_scales(const float* u, int width, const RowNorm& rn, float* scales) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  __shared__ float partial[32];
  if (rn.groups >= warps) {  // a warp takes whole parts
    for (int g = warp; g < rn.groups; g += warps) {
      float ss = 0.0f;
      for (int i = lane; i < rn.part; i += 32) ss += u[g * rn.part + i] * u[g * rn.part + i];
      ss = warp_sum(ss);
      if (lane == 0) scales[g] = 1.0f / sqrtf(ss / float(rn.part) + rn.n.eps);
    }
  } else {  // several warps share a part
    const int slices = warps / rn.groups, g = warp / slices, s = warp % slices;
    float ss = 0.0f;
    if (g < rn.groups)
      for (int i = s * 32 + lane; i < rn.part; i += 32 * slices) ss += u[g * rn.part + i] * u[g * rn.part + i];
    ss = warp_sum(ss);
    if (lane == 0) partial[warp] = ss;
    __syncthreads();
    if (threadIdx.x < rn.groups) {
      float t = 0.0f;
      for (int k = 0; k < slices; ++k) t += partial[threadIdx.x * slices + k];
      scales[threadIdx.x] = 1.0f / sqrtf(t / float(rn.part) + rn.n.eps);
    }
  }
  __syncthreads();
}

__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void put4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, const float4& v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

template <typename T, bool VEC>
__device__ __forceinline__ void store_normed(const float* u, int width, const RowNorm& rn, const float* scales, T* out) {
  const q38_norm& n = rn.n;
  if (VEC) {
    for (int c = 4 * threadIdx.x; c < width; c += 4 * blockDim.x) {
      const float4 v = *reinterpret_cast<const float4*>(u + c);
      const float s = scales[c / rn.part];  // parts are whole 16-byte pieces here
      const float4 g = n.gain_stride ? *reinterpret_cast<const float4*>(n.gain + c)
                                     : make_float4(n.gain[0], n.gain[0], n.gain[0], n.gain[0]);
      put4(out + c, make_float4(v.x * s * g.x, v.y * s * g.y, v.z * s * g.z, v.w * s * g.w));
    }
  } else {
    for (int c = threadIdx.x; c < width; c += blockDim.x) put(out + c, u[c] * scales[c / rn.part] * n.gain[c * n.gain_stride]);
  }
}

// ---- embedding ---------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(kMaxThreads)
stream_embed_kernel(const __nv_bfloat16* __restrict__ table, const int32_t* __restrict__ tokens, int width, float scale, int streams,
                    float* __restrict__ residual, const float* __restrict__ in, RowNorm rn, T* __restrict__ out, int ld) {
  extern __shared__ __align__(16) float sm[];
  float* u = sm;                           // [width rounded up to 4]
  float* scales = sm + (width + 3) / 4 * 4;  // [groups]
  float w = 0.0f;
  for (int s = 0; s < streams; ++s) w += in[s];  // all streams are equal here
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x;
  const __nv_bfloat16* e = table + (size_t)tokens[m] * width;
  float* x = residual + (size_t)m * streams * width;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float v = __bfloat162float(e[c]) * scale;
    for (int s = 0; s < streams; ++s) x[(size_t)s * width + c] = v;
    u[c] = w * v;
  }
  __syncthreads();
  part_scales(u, width, rn, scales);
  store_normed<T, false>(u, width, rn, scales, out + (size_t)m * ld);
}

// ---- update + next pre-norm ----------------------------------------------------------------------------------------------
// S = most streams this instance holds in registers.
template <typename T, int S, bool VEC>
__global__ void __launch_bounds__(kMaxThreads)
stream_norm_kernel(const float* __restrict__ y, int ldy, int width, int streams, q38_stream_update up, float* __restrict__ residual,
                   const float* __restrict__ in, RowNorm rn, T* __restrict__ out, int ld) {
  extern __shared__ __align__(16) float sm[];
  float* u = sm;
  float* scales = sm + (width + 3) / 4 * 4;
  __shared__ float mix[S][S], gain[S], take[S];
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) {
    const int a = i / S, b = i % S;
    mix[a][b] = a < streams && b < streams ? up.mix[a * streams + b] : 0.0f;
  }
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    gain[i] = i < streams ? up.mult * up.out[i] : 0.0f;
    take[i] = in && i < streams ? in[i] : 0.0f;
  }
  __syncthreads();
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x;
  const float* yr = y + (size_t)m * ldy;
  float* xr = residual + (size_t)m * streams * width;
  if (VEC) {
    for (int c = 4 * threadIdx.x; c < width; c += 4 * blockDim.x) {
      float4 x[S];
      const float4 v = *reinterpret_cast<const float4*>(yr + c);
#pragma unroll
      for (int s = 0; s < S; ++s)
        x[s] = s < streams ? *reinterpret_cast<const float4*>(xr + (size_t)s * width + c) : make_float4(0, 0, 0, 0);
      float4 sum = make_float4(0, 0, 0, 0);
#pragma unroll
      for (int t = 0; t < S; ++t) {
        if (t >= streams) break;
        float4 n = make_float4(gain[t] * v.x, gain[t] * v.y, gain[t] * v.z, gain[t] * v.w);
#pragma unroll
        for (int s = 0; s < S; ++s) {
          const float f = mix[s][t];
          n.x += f * x[s].x;
          n.y += f * x[s].y;
          n.z += f * x[s].z;
          n.w += f * x[s].w;
        }
        *reinterpret_cast<float4*>(xr + (size_t)t * width + c) = n;
        sum.x += take[t] * n.x;
        sum.y += take[t] * n.y;
        sum.z += take[t] * n.z;
        sum.w += take[t] * n.w;
      }
      *reinterpret_cast<float4*>(u + c) = sum;
    }
  } else {
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
      float x[S];
      const float v = yr[c];
#pragma unroll
      for (int s = 0; s < S; ++s) x[s] = s < streams ? xr[(size_t)s * width + c] : 0.0f;
      float sum = 0.0f;
#pragma unroll
      for (int t = 0; t < S; ++t) {
        if (t >= streams) break;
        float n = gain[t] * v;
#pragma unroll
        for (int s = 0; s < S; ++s) n += mix[s][t] * x[s];
        xr[(size_t)t * width + c] = n;
        sum += take[t] * n;
      }
      u[c] = sum;
    }
  }
  if (in == nullptr) return;
  __syncthreads();
  part_scales(u, width, rn, scales);
  store_normed<T, VEC>(u, width, rn, scales, out + (size_t)m * ld);
}

// ---- sum of the streams + final norm ---------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(kMaxThreads)
stream_gather_kernel(const float* __restrict__ residual, const int* __restrict__ rows, int first, int width, int streams, RowNorm rn,
                     T* __restrict__ out, int ld) {
  extern __shared__ __align__(16) float sm[];
  float* u = sm;
  float* scales = sm + (width + 3) / 4 * 4;
  pdl_wait();
  pdl_launch_dependents();
  const int src = rows ? rows[blockIdx.x] : first + int(blockIdx.x);
  const float* x = residual + (size_t)src * streams * width;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    float v = 0.0f;
    for (int s = 0; s < streams; ++s) v += x[(size_t)s * width + c];
    u[c] = v;
  }
  __syncthreads();
  part_scales(u, width, rn, scales);
  store_normed<T, false>(u, width, rn, scales, out + (size_t)blockIdx.x * ld);
}

// ---- launchers ----------------------------------------------------------------------------------------------------------------
struct Shape {
  int threads;
  size_t smem;
};
Shape shape_of(int m, int width, int groups) {
  // few rows: one 16-byte piece per thread; many: CTAs of 256 threads or fewer, several per SM
  const int most = m <= num_sms() ? kMaxThreads : 256;
  return {std::max(32, std::min(most, (width / 4 + 31) / 32 * 32)), (size_t((width + 3) / 4 * 4) + size_t(groups)) * 4};
}

int check_rows(const char* what, int m, int width, int streams, const q38_norm* n, const void* out, int ld, int act) {
  Q38_REQUIRE(m > 0 && width > 0 && streams > 0 && streams <= Q38_MAX_STREAMS, "%s: %d rows of %d streams of %d", what, m, streams, width);
  Q38_REQUIRE(act == Q38_ACT_BF16 || act == Q38_ACT_F32, "%s: activation precision %d", what, act);
  if (!n) return Q38_OK;
  const int groups = n->groups > 1 ? n->groups : 1;
  Q38_REQUIRE(n->gain && out && ld >= width, "%s: norm", what);
  Q38_REQUIRE(width % groups == 0 && (n->gain_stride == 0 || n->gain_stride == 1), "%s: %d parts of a row of %d", what, groups, width);
  Q38_REQUIRE(shape_of(m, width, groups).smem <= 48 * 1024, "%s: a row of %d with %d parts does not fit", what, width, groups);
  return Q38_OK;
}
RowNorm row_norm(const q38_norm& n, int width) {
  const int groups = n.groups > 1 ? n.groups : 1;
  return {n, groups, width / groups};
}
bool aligned16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

template <typename T, int S>
int launch_norm(const float* y, int ldy, int m, int width, int streams, const q38_stream_update& up, float* residual, const float* in,
                const RowNorm& rn, T* out, int ld, bool vec, cudaStream_t s) {
  const Shape sh = shape_of(m, width, rn.groups);
  if (S <= 4 && vec)
    (void)launch_kernel(stream_norm_kernel<T, S <= 4 ? S : 4, true>, dim3(m), dim3(sh.threads), sh.smem, s, y, ldy, width, streams, up,
                        residual, in, rn, out, ld);
  else
    (void)launch_kernel(stream_norm_kernel<T, S, false>, dim3(m), dim3(sh.threads), sh.smem, s, y, ldy, width, streams, up, residual, in,
                        rn, out, ld);
  Q38_LAUNCH_OK("stream_norm_kernel");
  return Q38_OK;
}

template <typename T>
int stream_norm(const float* y, int ldy, int m, int width, int streams, const q38_stream_update& up, float* residual, const float* in,
                const RowNorm& rn, T* out, int ld, cudaStream_t s) {
  const bool vec = width % 4 == 0 && ldy % 4 == 0 && aligned16(y) && aligned16(residual) &&
                   (!in || (ld % 4 == 0 && rn.part % 4 == 0 && aligned16(out) && aligned16(rn.n.gain)));
  if (streams == 1) return launch_norm<T, 1>(y, ldy, m, width, streams, up, residual, in, rn, out, ld, vec, s);
  if (streams == 2) return launch_norm<T, 2>(y, ldy, m, width, streams, up, residual, in, rn, out, ld, vec, s);
  if (streams <= 4) return launch_norm<T, 4>(y, ldy, m, width, streams, up, residual, in, rn, out, ld, vec, s);
  return launch_norm<T, Q38_MAX_STREAMS>(y, ldy, m, width, streams, up, residual, in, rn, out, ld, false, s);
}

}  // namespace
}  // namespace q38

using namespace q38;

extern "C" int q38_stream_embed(const q38_bf16* table, const int32_t* tokens, int m, int width, float scale, int streams,
                                float* residual, const float* in, const q38_norm* norm, void* out, int ld_out, int act,
                                void* stream) {
  if (m == 0) return Q38_OK;
  Q38_REQUIRE(table && tokens && residual && in && norm, "stream_embed: null argument");
  if (const int rc = check_rows("stream_embed", m, width, streams, norm, out, ld_out, act)) return rc;
  const RowNorm rn = row_norm(*norm, width);
  const Shape sh = shape_of(m, width, rn.groups);
  const auto* t = reinterpret_cast<const __nv_bfloat16*>(table);
  if (act == Q38_ACT_BF16)
    (void)launch_kernel(stream_embed_kernel<__nv_bfloat16>, dim3(m), dim3(sh.threads), sh.smem, as_stream(stream), t, tokens, width, scale,
                        streams, residual, in, rn, static_cast<__nv_bfloat16*>(out), ld_out);
  else
    (void)launch_kernel(stream_embed_kernel<float>, dim3(m), dim3(sh.threads), sh.smem, as_stream(stream), t, tokens, width, scale, streams,
                        residual, in, rn, static_cast<float*>(out), ld_out);
  Q38_LAUNCH_OK("stream_embed_kernel");
  return Q38_OK;
}

extern "C" int q38_stream_norm(const float* y, int ldy, int m, int width, int streams, const q38_stream_update* update,
                               float* residual, const float* in, const q38_norm* next, void* out, int ld_out, int act,
                               void* stream) {
  if (m == 0) return Q38_OK;
  Q38_REQUIRE(y && update && update->mix && update->out && residual && ldy >= width && (!next || in), "stream_norm: arguments");
  if (const int rc = check_rows("stream_norm", m, width, streams, next, out, ld_out, act)) return rc;
  const RowNorm rn = next ? row_norm(*next, width) : RowNorm{{nullptr, 0, 0.0f, 1}, 1, width};
  const float* take = next ? in : nullptr;
  return act == Q38_ACT_BF16 ? stream_norm(y, ldy, m, width, streams, *update, residual, take, rn, static_cast<__nv_bfloat16*>(out), ld_out,
                                           as_stream(stream))
                             : stream_norm(y, ldy, m, width, streams, *update, residual, take, rn, static_cast<float*>(out), ld_out,
                                           as_stream(stream));
}

extern "C" int q38_stream_gather(const float* residual, const int* rows, int first, int n, int width, int streams,
                                 const q38_norm* norm, void* out, int ld_out, int act, void* stream) {
  if (n == 0) return Q38_OK;
  Q38_REQUIRE(residual && norm && first >= 0, "stream_gather: arguments");
  if (const int rc = check_rows("stream_gather", n, width, streams, norm, out, ld_out, act)) return rc;
  const RowNorm rn = row_norm(*norm, width);
  const Shape sh = shape_of(n, width, rn.groups);
  if (act == Q38_ACT_BF16)
    (void)launch_kernel(stream_gather_kernel<__nv_bfloat16>, dim3(n), dim3(sh.threads), sh.smem, as_stream(stream), residual, rows, first,
                        width, streams, rn, static_cast<__nv_bfloat16*>(out), ld_out);
  else
    (void)launch_kernel(stream_gather_kernel<float>, dim3(n), dim3(sh.threads), sh.smem, as_stream(stream), residual, rows, first, width,
                        streams, rn, static_cast<float*>(out), ld_out);
  Q38_LAUNCH_OK("stream_gather_kernel");
  return Q38_OK;
}
