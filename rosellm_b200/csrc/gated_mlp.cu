// Elementwise steps of gated feed-forward layers.
//
// `gated_act_kernel`: the packed product [gate | up] of a token becomes f(gate, up) per unit
// (gated_act.cuh).  `token_gate_kernel`: a per-token input of a layer, out = gelu_tanh(s) * e
// with e the layer's part of the token's row in a second embedding table (the row is looked
// up by the token id here, so the part never exists as a tensor of its own).
#include "gated_act.cuh"
#include "gemm_vec.cuh"

namespace rl {

template <typename T, typename TOut>
__global__ void gated_act_kernel(const T* __restrict__ gu, long ld, int up_at, TOut* __restrict__ out, long ldo,
                                 int n_rows, int width, int kind, float alpha, float limit) {
  pdl_begin();
  const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long)n_rows * width) return;
  const int r = (int)(i / width), f = (int)(i - (long)r * width);
  const T* row = gu + (size_t)r * ld;
  out[(size_t)r * ldo + f] = from_f32<TOut>(gated_value(to_f32(row[f]), to_f32(row[up_at + f]), kind, alpha, limit));
}

__device__ __forceinline__ void load_eight(const float* p, float (&x)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  x[0] = a.x, x[1] = a.y, x[2] = a.z, x[3] = a.w, x[4] = b.x, x[5] = b.y, x[6] = b.z, x[7] = b.w;
}
__device__ __forceinline__ void load_eight(const __nv_bfloat16* p, float (&x)[8]) { Vec16<__nv_bfloat16>::load(p, x); }
__device__ __forceinline__ void store_eight(float* p, const float (&x)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(x[4], x[5], x[6], x[7]);
}
__device__ __forceinline__ void store_eight(__nv_bfloat16* p, const float (&x)[8]) {
  uint4 v;
  uint32_t* w = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 b = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
    w[i] = *reinterpret_cast<const uint32_t*>(&b);
  }
  *reinterpret_cast<uint4*>(p) = v;
}

// The same, eight units a thread (16-byte pieces): block (row, group of 8 * blockDim.x units).
template <typename T, typename TOut>
__global__ __launch_bounds__(256) void gated_act_vec_kernel(const T* __restrict__ gu, long ld, int up_at, TOut* __restrict__ out,
                                                            long ldo, int groups, int width, int kind, float alpha, float limit) {
  pdl_begin();
  const int r = blockIdx.x / groups, f = ((blockIdx.x - r * groups) * blockDim.x + threadIdx.x) * 8;
  if (f >= width) return;
  const T* row = gu + (size_t)r * ld + f;
  float g[8], u[8];
  load_eight(row, g);
  load_eight(row + up_at, u);
#pragma unroll
  for (int i = 0; i < 8; ++i) g[i] = gated_value(g[i], u[i], kind, alpha, limit);
  store_eight(out + (size_t)r * ldo + f, g);
}

template <typename T, typename TOut>
static void launch_gated_act(const void* gu, long ld, int up_at, void* out, long ldo, int n_rows, int width, int kind, float alpha,
                             float limit, cudaStream_t stream) {
  const bool vec = width % 8 == 0 && ld % 8 == 0 && up_at % 8 == 0 && ldo % 8 == 0 && (uintptr_t)gu % 16 == 0 && (uintptr_t)out % 16 == 0;
  if (vec) {
    int threads = (width / 8 + 31) / 32 * 32;
    threads = threads > 256 ? 256 : threads;
    const int groups = (width / 8 + threads - 1) / threads;
    launch_pdl(gated_act_vec_kernel<T, TOut>, (unsigned)((long)n_rows * groups), threads, 0, stream, (const T*)gu, ld, up_at, (TOut*)out,
               ldo, groups, width, kind, alpha, limit);
    return;
  }
  const long total = (long)n_rows * width;
  launch_pdl(gated_act_kernel<T, TOut>, (unsigned)((total + 255) / 256), 256, 0, stream, (const T*)gu, ld, up_at, (TOut*)out, ldo, n_rows,
             width, kind, alpha, limit);
}

// out[n, j] = gelu_tanh(s[n, j]) * table[id_n, col0 + j] for j < dim, 0 for dim <= j < out_width.
template <typename T>
__global__ void token_gate_kernel(const T* __restrict__ s, long lds, const int* __restrict__ ids,
                                  const T* __restrict__ table, long ldt, int col0, int dim, T* __restrict__ out,
                                  long ldo, int out_width, int n_tokens, int vocab, const int* __restrict__ feedback,
                                  int n_feedback, int* __restrict__ status) {
  pdl_begin();
  const int n = blockIdx.x;
  if (n >= n_tokens) return;
  int id = ids[n];
  if (id < 0 && feedback != nullptr && -id - 1 < n_feedback) id = feedback[-id - 1];
  const bool bad = id < 0 || id >= vocab;
  if (bad && threadIdx.x == 0) atomicOr(status, RL_STATUS_BAD_TOKEN);
  for (int j = threadIdx.x; j < out_width; j += blockDim.x) {
    float v = 0.f;
    if (j < dim && !bad) v = gelu_tanh_f32(to_f32(s[(size_t)n * lds + j])) * to_f32(table[(size_t)id * ldt + col0 + j]);
    out[(size_t)n * ldo + j] = from_f32<T>(v);
  }
}

}  // namespace rl

// gu: [rows, >= up_at + width] (row stride ld): gate at column f, up at column up_at + f.
// dtype, out_dtype: both the same, or float32 in and bfloat16 out.
RL_EXPORT int rl_gated_act(int dtype, int out_dtype, const void* gu, long ld, int up_at, void* out, long ldo, int n_rows,
                           int width, int kind, float alpha, float limit, cudaStream_t stream) {
  if (n_rows <= 0 || width <= 0) return 0;
  if (kind < 0 || kind > 3 || (dtype == RL_BF16 && out_dtype == RL_F32)) return -2;
  using bf16 = __nv_bfloat16;
  if (dtype == RL_F32 && out_dtype == RL_F32)
    rl::launch_gated_act<float, float>(gu, ld, up_at, out, ldo, n_rows, width, kind, alpha, limit, stream);
  else if (dtype == RL_F32)
    rl::launch_gated_act<float, bf16>(gu, ld, up_at, out, ldo, n_rows, width, kind, alpha, limit, stream);
  else
    rl::launch_gated_act<bf16, bf16>(gu, ld, up_at, out, ldo, n_rows, width, kind, alpha, limit, stream);
  RL_CHECK_LAUNCH();
  return 0;
}

RL_EXPORT int rl_token_gate(int dtype, const void* s, long lds, const int* ids, const void* table, long ldt, int col0,
                            int dim, void* out, long ldo, int out_width, int n_tokens, int vocab, const int* feedback,
                            int n_feedback, int* status, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (dim <= 0 || out_width < dim || status == nullptr) return -2;
  if (dtype == RL_F32)
    rl::launch_pdl(rl::token_gate_kernel<float>, n_tokens, 64, 0, stream, (const float*)s, lds, ids,
                   (const float*)table, ldt, col0, dim, (float*)out, ldo, out_width, n_tokens, vocab, feedback,
                   n_feedback, status);
  else
    rl::launch_pdl(rl::token_gate_kernel<__nv_bfloat16>, n_tokens, 64, 0, stream, (const __nv_bfloat16*)s, lds, ids,
                   (const __nv_bfloat16*)table, ldt, col0, dim, (__nv_bfloat16*)out, ldo, out_width, n_tokens, vocab,
                   feedback, n_feedback, status);
  RL_CHECK_LAUNCH();
  return 0;
}
