// parallel_ops.cu — elementwise kernels of the parallel layer form whose sublayers share ONE norm (h = N x,
// x <- x + mixer(h) + ff(h)):
//
//   layer_close:  x += y + bias;  out = N(x)       the sum that closes a layer and the norm that opens the next, one pass;
//                                                  y is a row of the product, or its split-K partial sums in fp32
//   clamped_glu:  y = g' sigmoid(1.702 g') (u' + 1), g' = min(g + bg, limit), u' = clamp(u + bu, -limit, limit)
//                 over strided rows whose gate and up columns lie side by side or interleaved in blocks
//
// N is the zero-centred RMS norm, x / sqrt(mean(x^2) + eps) * (1 + w).  All arithmetic is fp32; only y (unless partial
// sums), out and the unit's rows are in the model dtype.
#include <algorithm>

#include "layered_common.cuh"

namespace b200q {

template <typename T> __device__ __forceinline__ void get4(const T* p, float (&v)[4]);
template <> __device__ __forceinline__ void get4<float>(const float* p, float (&v)[4]) {
  const float4 f = *reinterpret_cast<const float4*>(p);
  v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
template <> __device__ __forceinline__ void get4<bf16>(const bf16* p, float (&v)[4]) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  v[0] = bf16_lo(u.x); v[1] = bf16_hi(u.x); v[2] = bf16_lo(u.y); v[3] = bf16_hi(u.y);
}
template <typename T> __device__ __forceinline__ void put4(T* p, const float (&v)[4]);
template <> __device__ __forceinline__ void put4<float>(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void put4<bf16>(bf16* p, const float (&v)[4]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
}

// CTA per row.  Rows of up to 256 * 4 * CLOSE_KEEP values whose width is a multiple of 4 stay in registers between the
// sum and the norm; other rows are read back.  Partial sums are added in split order.
constexpr int CLOSE_KEEP = 8;
template <typename TY, typename T>
__global__ void __launch_bounds__(256) layer_close_kernel(float* __restrict__ x, const TY* __restrict__ y, int splits,
                                                          long long split_stride, const float* __restrict__ bias,
                                                          const float* __restrict__ w, T* __restrict__ out, int W, float eps,
                                                          int vec) {
  __shared__ float red[32];
  const long long base = (long long)blockIdx.x * W;
  float ss = 0.f;
  if (vec) {
    float v[CLOSE_KEEP][4];
#pragma unroll
    for (int q = 0; q < CLOSE_KEEP; ++q) {
      const int c = (q * 256 + threadIdx.x) * 4;
      if (c >= W) continue;
      float a[4], b[4];
      get4(y + base + c, a);
      for (int s = 1; s < splits; ++s) {
        get4(y + s * split_stride + base + c, b);
#pragma unroll
        for (int i = 0; i < 4; ++i) a[i] += b[i];
      }
      if (bias) {
        get4(bias + c, b);
#pragma unroll
        for (int i = 0; i < 4; ++i) a[i] += b[i];
      }
      get4(x + base + c, b);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[q][i] = a[i] + b[i];
        ss = fmaf(v[q][i], v[q][i], ss);
      }
      put4(x + base + c, v[q]);
    }
    if (!out) return;
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)W + eps);
#pragma unroll
    for (int q = 0; q < CLOSE_KEEP; ++q) {
      const int c = (q * 256 + threadIdx.x) * 4;
      if (c >= W) continue;
      float n[4];
      get4(w + c, n);
#pragma unroll
      for (int i = 0; i < 4; ++i) n[i] = v[q][i] * inv * (1.f + n[i]);
      put4(out + base + c, n);
    }
    return;
  }
  for (int c = threadIdx.x; c < W; c += 256) {
    float a = ldf(y + base + c);
    for (int s = 1; s < splits; ++s) a += ldf(y + s * split_stride + base + c);
    if (bias) a += bias[c];
    a += x[base + c];
    x[base + c] = a;
    ss = fmaf(a, a, ss);
  }
  if (!out) return;
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)W + eps);
  for (int c = threadIdx.x; c < W; c += 256) stf(out + base + c, x[base + c] * inv * (1.f + w[c]));
}

__device__ __forceinline__ float clamped_unit(float g, float u, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoidf_(1.702f * g) * (u + 1.f);
}

// where column c's gate lies in a row (block 0: [g (F) | u (F)], block b: interleaved in blocks of b); up = gate + step
__device__ __forceinline__ int gate_column(int c, int block) { return block > 0 ? (c / block) * 2 * block + c % block : c; }

template <typename T>
__global__ void __launch_bounds__(256) clamped_glu_ex_kernel(const T* __restrict__ gu, int ld_in,
                                                             const float* __restrict__ bias, T* __restrict__ y, int ld_out,
                                                             long long rows, int F, int block, float limit) {
  const long long total = rows * F;
  const int step = block > 0 ? block : F;
  for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total;
       e += (long long)gridDim.x * blockDim.x) {
    const long long r = e / F;
    const int c = (int)(e % F), ga = gate_column(c, block);
    float g = ldf(gu + r * ld_in + ga), u = ldf(gu + r * ld_in + ga + step);
    if (bias) {
      g += bias[ga];
      u += bias[ga + step];
    }
    stf(y + r * ld_out + c, clamped_unit(g, u, limit));
  }
}
__global__ void __launch_bounds__(256) clamped_glu_ex_v8_kernel(const bf16* __restrict__ gu, int ld_in,
                                                                const float* __restrict__ bias, bf16* __restrict__ y,
                                                                int ld_out, long long rows, int F, int block, float limit) {
  const int per = F / 8, step = block > 0 ? block : F;
  const long long total = rows * per;
  for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total;
       e += (long long)gridDim.x * blockDim.x) {
    const long long r = e / per;
    const int c = (int)(e % per) * 8, ga = gate_column(c, block);  // block is a multiple of 8: eight columns stay together
    const uint4 g4 = ld_v4(gu + r * ld_in + ga), u4 = ld_v4(gu + r * ld_in + ga + step);
    const uint32_t gw[4] = {g4.x, g4.y, g4.z, g4.w}, uw[4] = {u4.x, u4.y, u4.z, u4.w};
    float g[8], u[8];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      g[2 * i] = bf16_lo(gw[i]);
      g[2 * i + 1] = bf16_hi(gw[i]);
      u[2 * i] = bf16_lo(uw[i]);
      u[2 * i + 1] = bf16_hi(uw[i]);
    }
    if (bias) {
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        float a[4], b[4];
        get4(bias + ga + 4 * q, a);
        get4(bias + ga + step + 4 * q, b);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          g[4 * q + i] += a[i];
          u[4 * q + i] += b[i];
        }
      }
    }
    uint32_t o[4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
      o[i] = pack_bf16x2(clamped_unit(g[2 * i], u[2 * i], limit), clamped_unit(g[2 * i + 1], u[2 * i + 1], limit));
    st_v4(y + r * ld_out + c, make_uint4(o[0], o[1], o[2], o[3]));
  }
}

}  // namespace b200q

using namespace b200q;

extern "C" {

int b200q_layer_close(float* x, const void* y, int y_f32, int splits, const float* bias, const float* w, void* out, int T_,
                      int W, float eps, int dtype, void* stream) {
  B200Q_CHECK_ARG(x && y && splits > 0 && (!out || w) && T_ >= 0 && W > 0 && is_dtype(dtype) &&
                      (splits == 1 || y_f32 || dtype == B200Q_DTYPE_F32),
                  "layer_close: bad argument (W=%d splits=%d)", W, splits);
  if (T_ == 0) return B200Q_OK;
  const int vec = W % 4 == 0 && W <= 256 * 4 * CLOSE_KEEP &&
                          ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(bias) |
                            reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out)) & 15) == 0
                      ? 1
                      : 0;
  const long long stride = (long long)T_ * W;
  cudaStream_t st = as_stream(stream);
  if (y_f32)
    DISPATCH_T(dtype, (layer_close_kernel<float, T><<<T_, 256, 0, st>>>(x, (const float*)y, splits, stride, bias, w, (T*)out, W,
                                                                        eps, vec)));
  else
    DISPATCH_T(dtype, (layer_close_kernel<T, T><<<T_, 256, 0, st>>>(x, (const T*)y, splits, stride, bias, w, (T*)out, W, eps,
                                                                    vec)));
  B200Q_LAUNCH_CHECK();
  return B200Q_OK;
}

int b200q_clamped_glu_ex(const void* gate_up, int ld_in, const float* bias, void* y, int ld_out, int64_t rows, int F, int block,
                         float limit, int dtype, void* stream) {
  B200Q_CHECK_ARG(gate_up && y && rows >= 0 && F > 0 && ld_in >= 2 * F && ld_out >= F && block >= 0 &&
                      (block == 0 || F % block == 0) && limit >= 0.f && is_dtype(dtype),
                  "clamped_glu: bad argument (F=%d, blocks of %d, rows of %d and %d)", F, block, ld_in, ld_out);
  if (rows == 0) return B200Q_OK;
  cudaStream_t st = as_stream(stream);
  if (dtype == B200Q_DTYPE_BF16 && F % 8 == 0 && block % 8 == 0 && ld_in % 8 == 0 && ld_out % 8 == 0 &&
      ((reinterpret_cast<uintptr_t>(gate_up) | reinterpret_cast<uintptr_t>(bias) | reinterpret_cast<uintptr_t>(y)) & 15) == 0)
    clamped_glu_ex_v8_kernel<<<grid_for(rows * (F / 8)), 256, 0, st>>>((const bf16*)gate_up, ld_in, bias, (bf16*)y, ld_out,
                                                                       rows, F, block, limit);
  else
    DISPATCH_T(dtype, (clamped_glu_ex_kernel<T><<<grid_for(rows * F), 256, 0, st>>>((const T*)gate_up, ld_in, bias, (T*)y,
                                                                                    ld_out, rows, F, block, limit)));
  B200Q_LAUNCH_CHECK();
  return B200Q_OK;
}

}  // extern "C"
