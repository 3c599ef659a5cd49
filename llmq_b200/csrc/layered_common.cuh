// layered_common.cuh — device helpers shared by the kernels of the layered architectures
// (layered_ops.cu, sequence_ops.cu): typed loads / stores over the model's element type, block
// reductions with a fixed summation order, and the dtype dispatch of the entry points.
#pragma once
#include "common.cuh"

namespace b200q {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<bf16>(const bf16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void stf(T* p, float v);
template <> __device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void stf<bf16>(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// sum over the block (blockDim.x a multiple of 32, <= 1024); red: >= 32 floats of shared memory.
// Every thread adds the warp partials in the same order, so all threads hold the same bits.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
  __syncthreads();
  if (lane == 0) red[w] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < nw; ++i) t += red[i];
  return t;
}
__device__ __forceinline__ float sigmoidf_(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float siluf_(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplusf_(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// ---- bounded wait on an mbarrier: false when it ran out (about two seconds), so that a kernel can give up ----
__device__ __forceinline__ bool mbar_wait_limited(uint64_t* bar, uint32_t parity) {
  const long long t0 = clock64();
  for (int i = 0; i < (1 << 26); ++i) {
    if (mbar_try_wait(bar, parity)) return true;
    if (clock64() - t0 > 4000000000ll) break;
  }
  return false;
}
int* wait_flag(int** dev);  // where such a kernel says so (diff_attn.cu): host and device address of one int

static inline int grid_for(long long total, int block = 256) {
  long long g = (total + block - 1) / block;
  return (int)(g < 1 ? 1 : (g > 148 * 16 ? 148 * 16 : g));
}
// portion_attn.cu: grouped-query attention of a step's portions and single tokens on the tensor cores (behind b200q_window_attn_sink)
bool portion_attn_gqa_ok(const float* qs, const void* cache, const void* out, int kv_heads, int dim, int vdim, int block_size);
int portion_attn_gqa(const float* qs, const void* cache, const int32_t* block_table, int bt_stride, const int32_t* seq_desc,
                     int n_seqs, int longest, int T, int heads, int kv_heads, int dim, int vdim, int block_size, int window,
                     const float* sink, const void* gate, int ld_gate, int channel_gate, void* out, cudaStream_t st);
// ... and attention in the latent space (behind b200q_latent_attn_sink)
bool latent_tokens_ok(const float* qa, const void* cache, const void* out, int R, int P, int block_size);
int latent_tokens(const float* qa, const void* cache, const int32_t* block_table, int bt_stride, const int32_t* row_seq,
                  const int32_t* positions, int T, int heads, int R, int P, int block_size, int window, float scale,
                  const float* sink, const void* gate, int ld_gate, void* out, cudaStream_t st);

static inline bool is_dtype(int d) { return d == B200Q_DTYPE_BF16 || d == B200Q_DTYPE_F32; }

}  // namespace b200q

#define DISPATCH_T(dtype, ...)                   \
  do {                                           \
    if ((dtype) == B200Q_DTYPE_F32) {            \
      using T = float;                           \
      __VA_ARGS__;                               \
    } else {                                     \
      using T = bf16;                            \
      __VA_ARGS__;                               \
    }                                            \
  } while (0)
