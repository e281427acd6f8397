// RMS norm: y = x / sqrt(mean(x^2) + eps) * w, statistics and arithmetic in float32.
//
// Two uses.  `rmsnorm_store_kernel` writes normalised rows (optionally gathered by index) in
// float32 or bfloat16: a final norm ahead of a head, or a norm ahead of a sublayer.
// `rmsnorm_add_kernel` serves blocks that normalise a sublayer's OUTPUT: the float32 residual
// stream gets `stream += mult * rmsnorm(y) * w`, and the same kernel may leave a bfloat16 copy
// of the stream's new rows for the products of the next sublayer to read, so that no kernel of
// its own has to round the stream.  `cast_rows_kernel` makes that copy where nothing precedes.
#include "common.cuh"

namespace rl {

// One block per row; the row is read twice (the second time from L1/L2).
template <typename TOut>
__global__ __launch_bounds__(256) void rmsnorm_store_kernel(const float* __restrict__ x, long ldx,
                                                            const int* __restrict__ rows,
                                                            const float* __restrict__ gamma, TOut* __restrict__ out,
                                                            long ldo, int n_out, int width, float eps) {
  __shared__ float scratch[33];
  pdl_begin();
  const int i = blockIdx.x;
  if (i >= n_out) return;
  const int src = rows != nullptr ? rows[i] : i;
  const float* xr = x + (size_t)src * ldx;
  float s = 0.f;
  for (int d = threadIdx.x; d < width; d += blockDim.x) {
    const float v = xr[d];
    s = fmaf(v, v, s);
  }
  const float r = 1.0f / sqrtf(block_sum(s, scratch) / (float)width + eps);
  TOut* o = out + (size_t)i * ldo;
  for (int d = threadIdx.x; d < width; d += blockDim.x) o[d] = from_f32<TOut>(xr[d] * r * gamma[d]);
}

// stream[i] += mult * rmsnorm(y[i]) * gamma; copy[i] = bfloat16(stream[i]) when copy is given.
// VEC: widths and row strides are multiples of 4 and every row starts on a 16-byte boundary
// (8-byte for the copy): 16-byte loads and stores.
template <bool VEC>
__global__ __launch_bounds__(256) void rmsnorm_add_kernel(const float* __restrict__ y, long ldy,
                                                          const float* __restrict__ gamma, float* __restrict__ stream,
                                                          long lds, __nv_bfloat16* __restrict__ copy, long ldc,
                                                          int n_rows, int width, float eps, float mult) {
  __shared__ float scratch[33];
  pdl_begin();
  const int i = blockIdx.x;
  if (i >= n_rows) return;
  const float* yr = y + (size_t)i * ldy;
  float* xr = stream + (size_t)i * lds;
  float s = 0.f;
  if (VEC) {
    const float4* y4 = reinterpret_cast<const float4*>(yr);
    for (int d = threadIdx.x; d < width / 4; d += blockDim.x) {
      const float4 v = y4[d];
      s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
    }
  } else {
    for (int d = threadIdx.x; d < width; d += blockDim.x) s = fmaf(yr[d], yr[d], s);
  }
  const float r = 1.0f / sqrtf(block_sum(s, scratch) / (float)width + eps);
  if (VEC) {
    const float4* y4 = reinterpret_cast<const float4*>(yr);
    const float4* g4 = reinterpret_cast<const float4*>(gamma);
    float4* x4 = reinterpret_cast<float4*>(xr);
    for (int d = threadIdx.x; d < width / 4; d += blockDim.x) {
      const float4 v = y4[d], g = g4[d];
      float4 x = x4[d];
      x.x += mult * (v.x * r * g.x);
      x.y += mult * (v.y * r * g.y);
      x.z += mult * (v.z * r * g.z);
      x.w += mult * (v.w * r * g.w);
      x4[d] = x;
      if (copy != nullptr) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(x.x, x.y), hi = __floats2bfloat162_rn(x.z, x.w);
        uint2 packed;
        packed.x = *reinterpret_cast<const uint32_t*>(&lo);
        packed.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(copy + (size_t)i * ldc + 4 * d) = packed;
      }
    }
  } else {
    for (int d = threadIdx.x; d < width; d += blockDim.x) {
      const float v = xr[d] + mult * (yr[d] * r * gamma[d]);
      xr[d] = v;
      if (copy != nullptr) copy[(size_t)i * ldc + d] = __float2bfloat16_rn(v);
    }
  }
}

// stream[i] += rmsnorm(y[i]) * gamma, and next[i] = rmsnorm(stream[i]) * gamma_next of the new row, in one
// pass: the norm after one sublayer and the norm before the next (a layer that normalises its sublayers on
// both sides).  The row is kept in shared memory between the two statistics.
template <typename TOut>
__global__ __launch_bounds__(256) void rmsnorm_add_norm_kernel(const float* __restrict__ y, long ldy,
                                                               const float* __restrict__ gamma,
                                                               float* __restrict__ stream, long lds,
                                                               const float* __restrict__ gamma_next,
                                                               TOut* __restrict__ next, long ldn, int n_rows, int width,
                                                               float eps, float eps_next) {
  extern __shared__ float row_s[];  // [width] + 33
  float* scratch = row_s + width;
  pdl_begin();
  const int i = blockIdx.x;
  if (i >= n_rows) return;
  const float* yr = y + (size_t)i * ldy;
  float* xr = stream + (size_t)i * lds;
  float s = 0.f;
  for (int d = threadIdx.x; d < width; d += blockDim.x) {
    const float v = yr[d];
    row_s[d] = v;
    s = fmaf(v, v, s);
  }
  const float r = 1.0f / sqrtf(block_sum(s, scratch) / (float)width + eps);
  float s2 = 0.f;
  for (int d = threadIdx.x; d < width; d += blockDim.x) {
    const float v = xr[d] + row_s[d] * r * gamma[d];
    xr[d] = v;
    row_s[d] = v;
    s2 = fmaf(v, v, s2);
  }
  const float r2 = 1.0f / sqrtf(block_sum(s2, scratch) / (float)width + eps_next);
  TOut* o = next + (size_t)i * ldn;
  for (int d = threadIdx.x; d < width; d += blockDim.x) o[d] = from_f32<TOut>(row_s[d] * r2 * gamma_next[d]);
}

// What a sublayer gave, row by row: y itself, or (y null) a mixture of experts not yet summed: sum_j weights[t, j] *
// eo[place_of[t, j]] + shared[t] * sigmoid(sg[t]) (weights, shared, sg may be null: factors of 1, nothing added), in
// moe_combine_kernel's order.
struct SublayerRows {
  const float* y;
  long ldy;
  const float* eo;
  const float* weights;
  const int* place_of;
  int top;
  const float* shared;
  long ldshared;
  const float* sg;
  long ldsg;
};

// The same two norms with everything a row needs in flight at once: a thread keeps its KEEP pieces of four entries of the
// sublayer's row, the stream's row and both norms' weights in registers (the weights are fetched before the wait for the
// kernels ahead), and the sum over a token's experts is formed on the way in (fused: no combine kernel, no buffer of
// summed rows).  NEXT off: the addition to the stream alone.
template <typename TOut, int KEEP, bool EXPERTS, bool NEXT>
__global__ __launch_bounds__(256) void rmsnorm_add_norm_vec_kernel(const SublayerRows src, const float* __restrict__ gamma,
                                                                   float* __restrict__ stream, long lds,
                                                                   const float* __restrict__ gamma_next, TOut* __restrict__ next,
                                                                   long ldn, int width, float eps, float eps_next) {
  __shared__ float scratch[33];
  const int i = blockIdx.x, pieces = width / 4;
  float4 y[KEEP], x[KEEP], g[KEEP], gn[KEEP];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int d = threadIdx.x + k * blockDim.x;
    g[k] = d < pieces ? reinterpret_cast<const float4*>(gamma)[d] : zero;
    if (NEXT) gn[k] = d < pieces ? reinterpret_cast<const float4*>(gamma_next)[d] : zero;
  }
  asm volatile("griddepcontrol.wait;" ::: "memory");
  float4* xr = reinterpret_cast<float4*>(stream + (size_t)i * lds);
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int d = threadIdx.x + k * blockDim.x;
    x[k] = d < pieces ? xr[d] : zero;
    if (EXPERTS) y[k] = zero;
    else y[k] = d < pieces ? reinterpret_cast<const float4*>(src.y + (size_t)i * src.ldy)[d] : zero;
  }
  if (EXPERTS) {
    auto add = [&](float w, const float* row) {
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int d = threadIdx.x + k * blockDim.x;
        if (d < pieces) {
          const float4 v = reinterpret_cast<const float4*>(row)[d];
          y[k].x = fmaf(w, v.x, y[k].x);
          y[k].y = fmaf(w, v.y, y[k].y);
          y[k].z = fmaf(w, v.z, y[k].z);
          y[k].w = fmaf(w, v.w, y[k].w);
        }
      }
    };
#pragma unroll 4
    for (int j = 0; j < src.top; ++j) {
      const size_t at = (size_t)i * src.top + j;
      add(src.weights != nullptr ? src.weights[at] : 1.f, src.eo + (size_t)src.place_of[at] * width);
    }
    if (src.shared != nullptr)
      add(src.sg != nullptr ? 1.0f / (1.0f + expf(-src.sg[(size_t)i * src.ldsg])) : 1.f, src.shared + (size_t)i * src.ldshared);
  }
  float s = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) s = fmaf(y[k].x, y[k].x, fmaf(y[k].y, y[k].y, fmaf(y[k].z, y[k].z, fmaf(y[k].w, y[k].w, s))));
  const float r = 1.0f / sqrtf(block_sum(s, scratch) / (float)width + eps);
  float s2 = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int d = threadIdx.x + k * blockDim.x;
    x[k].x += y[k].x * r * g[k].x;
    x[k].y += y[k].y * r * g[k].y;
    x[k].z += y[k].z * r * g[k].z;
    x[k].w += y[k].w * r * g[k].w;
    if (d < pieces) xr[d] = x[k];
    s2 = fmaf(x[k].x, x[k].x, fmaf(x[k].y, x[k].y, fmaf(x[k].z, x[k].z, fmaf(x[k].w, x[k].w, s2))));
  }
  if (!NEXT) return;
  const float r2 = 1.0f / sqrtf(block_sum(s2, scratch) / (float)width + eps_next);
  TOut* o = next + (size_t)i * ldn;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int d = threadIdx.x + k * blockDim.x;
    if (d >= pieces) continue;
    const float4 v = make_float4(x[k].x * r2 * gn[k].x, x[k].y * r2 * gn[k].y, x[k].z * r2 * gn[k].z, x[k].w * r2 * gn[k].w);
    if (sizeof(TOut) == 4) {
      reinterpret_cast<float4*>(o)[d] = v;
    } else {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
      reinterpret_cast<uint2*>(o)[d] = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    }
  }
}

__global__ void cast_rows_kernel(const float* __restrict__ x, __nv_bfloat16* __restrict__ out, long n) {
  pdl_begin();
  const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) out[i] = __float2bfloat16_rn(x[i]);
}

// stream[i] = rmsnorm(alpha * stream[i] + sigmoid(z[i] + zb) * (s0 * y0[i] + s1 * y1[i])) * gamma: the norm AFTER the sum
// of a layer that normalises the stream itself, with the sublayer's result (of one mixer, or of two side by
// side with a weight each) passing a gate whose logits z the caller computed from the sublayer's input (zb: the
// logits' bias, one entry a column, where the product that made z did not add it; null: none).  The new
// row also goes out in bfloat16 (copy) for the products of the next sublayer.  The row is kept in shared memory
// between the statistic and the scaling where it fits (KEEP), else worked out a second time.
template <bool KEEP>
__global__ __launch_bounds__(256) void gated_join_norm_kernel(const float* __restrict__ y0, long ld0, float s0,
                                                              const float* __restrict__ y1, long ld1, float s1,
                                                              const float* __restrict__ z, long ldz,
                                                              const float* __restrict__ zb,
                                                              const float* __restrict__ gamma, float* __restrict__ stream,
                                                              long lds, __nv_bfloat16* __restrict__ copy, long ldc,
                                                              int n_rows, int width, float eps, float alpha) {
  extern __shared__ float join_row_s[];
  __shared__ float scratch[33];
  pdl_begin();
  const int i = blockIdx.x;
  if (i >= n_rows) return;
  float* xr = stream + (size_t)i * lds;
  const float* a = y0 + (size_t)i * ld0;
  const float* b = y1 != nullptr ? y1 + (size_t)i * ld1 : nullptr;
  const float* zr = z != nullptr ? z + (size_t)i * ldz : nullptr;  // no logits: no gate
  auto joined = [&](int d) {
    float y = s0 * a[d];
    if (b != nullptr) y = fmaf(s1, b[d], y);
    const float g = zr != nullptr ? 1.0f / (1.0f + expf(-(zr[d] + (zb != nullptr ? zb[d] : 0.f)))) : 1.0f;
    return fmaf(alpha, xr[d], g * y);
  };
  float ss = 0.f;
  for (int d = threadIdx.x; d < width; d += blockDim.x) {
    const float v = joined(d);
    if (KEEP) join_row_s[d] = v;
    ss = fmaf(v, v, ss);
  }
  const float r = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
  for (int d = threadIdx.x; d < width; d += blockDim.x) {  // a thread meets the entries it wrote itself
    const float v = (KEEP ? join_row_s[d] : joined(d)) * r * gamma[d];
    xr[d] = v;
    if (copy != nullptr) copy[(size_t)i * ldc + d] = __float2bfloat16_rn(v);
  }
}

static inline int norm_threads(int width) {
  int t = (width + 3) / 4;
  t = (t + 31) / 32 * 32;
  return t < 32 ? 32 : (t > 256 ? 256 : t);
}

constexpr int RMS_VEC_MAX_WIDTH = 4 * 4 * 256;  // four pieces of four entries for each of 256 threads

template <typename TOut, bool EXPERTS, bool NEXT>
static void launch_add_norm_vec(const SublayerRows& src, const float* gamma, float* stream_rows, long lds, const float* gamma_next,
                                TOut* next, long ldn, int n_rows, int width, float eps, float eps_next, cudaStream_t stream) {
  const int pieces = width / 4;
  int threads = (pieces + 31) / 32 * 32;
  threads = threads > 256 ? 256 : threads;
  auto kernel = pieces <= threads ? rmsnorm_add_norm_vec_kernel<TOut, 1, EXPERTS, NEXT>
                                  : (pieces <= 2 * threads ? rmsnorm_add_norm_vec_kernel<TOut, 2, EXPERTS, NEXT>
                                                           : rmsnorm_add_norm_vec_kernel<TOut, 4, EXPERTS, NEXT>);
  launch_pdl(kernel, n_rows, threads, 0, stream, src, gamma, stream_rows, lds, gamma_next, next, ldn, width, eps, eps_next);
}

}  // namespace rl

// out[i] = rmsnorm(x[rows[i]] or x[i]) * gamma.  out_dtype: RL_F32 or RL_BF16.
RL_EXPORT int rl_rmsnorm(int out_dtype, const float* x, long ldx, const int* rows, const float* gamma, void* out,
                         long ldo, int n_out, int width, float eps, cudaStream_t stream) {
  if (n_out <= 0) return 0;
  if (width <= 0) return -2;
  const int threads = rl::norm_threads(width);
  if (out_dtype == RL_F32)
    rl::launch_pdl(rl::rmsnorm_store_kernel<float>, n_out, threads, 0, stream, x, ldx, rows, gamma, (float*)out, ldo,
                   n_out, width, eps);
  else
    rl::launch_pdl(rl::rmsnorm_store_kernel<__nv_bfloat16>, n_out, threads, 0, stream, x, ldx, rows, gamma,
                   (__nv_bfloat16*)out, ldo, n_out, width, eps);
  RL_CHECK_LAUNCH();
  return 0;
}

// stream += mult * rmsnorm(y) * gamma, with an optional bfloat16 copy of the stream's new rows.
RL_EXPORT int rl_rmsnorm_add(const float* y, long ldy, const float* gamma, float* stream_rows, long lds, void* copy,
                             long ldc, int n_rows, int width, float eps, float mult, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (width <= 0) return -2;
  const bool vec = width % 4 == 0 && ldy % 4 == 0 && lds % 4 == 0 && ldc % 4 == 0 && (uintptr_t)y % 16 == 0 &&
                   (uintptr_t)stream_rows % 16 == 0 && (uintptr_t)gamma % 16 == 0 && (uintptr_t)copy % 8 == 0;
  rl::launch_pdl(vec ? rl::rmsnorm_add_kernel<true> : rl::rmsnorm_add_kernel<false>, n_rows, rl::norm_threads(width), 0,
                 stream, y, ldy, gamma, stream_rows, lds, (__nv_bfloat16*)copy, ldc, n_rows, width, eps, mult);
  RL_CHECK_LAUNCH();
  return 0;
}

// out = bfloat16(x), n elements.
RL_EXPORT int rl_cast_rows(const float* x, void* out, long n, cudaStream_t stream) {
  if (n <= 0) return 0;
  rl::launch_pdl(rl::cast_rows_kernel, (unsigned)((n + 255) / 256), 256, 0, stream, x, (__nv_bfloat16*)out, n);
  RL_CHECK_LAUNCH();
  return 0;
}

// stream += rmsnorm(y) * gamma; next = rmsnorm(new stream rows) * gamma_next (out_dtype: RL_F32 or RL_BF16).
RL_EXPORT int rl_rmsnorm_add_norm(int out_dtype, const float* y, long ldy, const float* gamma, float* stream_rows,
                                  long lds, const float* gamma_next, void* next, long ldn, int n_rows, int width,
                                  float eps, float eps_next, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (width <= 0 || width > 48 * 1024 / 4 - 64) return -2;
  const int osize = out_dtype == RL_F32 ? 4 : 2;
  if (width % 4 == 0 && width <= rl::RMS_VEC_MAX_WIDTH && ldy % 4 == 0 && lds % 4 == 0 && ldn % 4 == 0 && (uintptr_t)y % 16 == 0 &&
      (uintptr_t)stream_rows % 16 == 0 && (uintptr_t)gamma % 16 == 0 && (uintptr_t)gamma_next % 16 == 0 &&
      (uintptr_t)next % (4 * osize) == 0) {
    const rl::SublayerRows src{y, ldy};
    if (out_dtype == RL_F32)
      rl::launch_add_norm_vec<float, false, true>(src, gamma, stream_rows, lds, gamma_next, (float*)next, ldn, n_rows, width, eps,
                                                  eps_next, stream);
    else
      rl::launch_add_norm_vec<__nv_bfloat16, false, true>(src, gamma, stream_rows, lds, gamma_next, (__nv_bfloat16*)next, ldn, n_rows,
                                                          width, eps, eps_next, stream);
    RL_CHECK_LAUNCH();
    return 0;
  }
  const size_t smem = (size_t)(width + 33) * sizeof(float);
  if (out_dtype == RL_F32)
    rl::launch_pdl(rl::rmsnorm_add_norm_kernel<float>, n_rows, rl::norm_threads(width), smem, stream, y, ldy, gamma,
                   stream_rows, lds, gamma_next, (float*)next, ldn, n_rows, width, eps, eps_next);
  else
    rl::launch_pdl(rl::rmsnorm_add_norm_kernel<__nv_bfloat16>, n_rows, rl::norm_threads(width), smem, stream, y, ldy,
                   gamma, stream_rows, lds, gamma_next, (__nv_bfloat16*)next, ldn, n_rows, width, eps, eps_next);
  RL_CHECK_LAUNCH();
  return 0;
}

// 1 if rl_rmsnorm_add_experts takes rows of this width.
RL_EXPORT int rl_rmsnorm_add_experts_fits(int width) { return width > 0 && width % 4 == 0 && width <= rl::RMS_VEC_MAX_WIDTH; }

// The same (next null: without the second norm) for a mixture of experts not yet summed: y[t] = sum_j weights[t, j] *
// eo[place_of[t, j]] + shared[t] * sigmoid(sg[t]); eo float32 [pairs, width], the rest as rl_moe_experts takes it.  Rows in
// 16-byte pieces.
RL_EXPORT int rl_rmsnorm_add_experts(int out_dtype, const float* eo, const float* weights, const int* place_of, int top,
                                     const float* shared, long ldshared, const float* sg, long ldsg, const float* gamma,
                                     float* stream_rows, long lds, const float* gamma_next, void* next, long ldn, int n_rows,
                                     int width, float eps, float eps_next, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  const int osize = out_dtype == RL_F32 ? 4 : 2;
  if (!rl_rmsnorm_add_experts_fits(width) || top <= 0 || (shared == nullptr && sg != nullptr) || (next != nullptr && gamma_next == nullptr) ||
      ldshared % 4 != 0 || lds % 4 != 0 || ldn % 4 != 0 ||
      (((uintptr_t)eo | (uintptr_t)shared | (uintptr_t)gamma | (uintptr_t)gamma_next | (uintptr_t)stream_rows) % 16) != 0 ||
      (uintptr_t)next % (4 * osize) != 0)
    return -2;
  const rl::SublayerRows src{nullptr, 0, eo, weights, place_of, top, shared, ldshared, sg, ldsg};
  if (next == nullptr)
    rl::launch_add_norm_vec<float, true, false>(src, gamma, stream_rows, lds, nullptr, nullptr, 0, n_rows, width, eps, eps_next, stream);
  else if (out_dtype == RL_F32)
    rl::launch_add_norm_vec<float, true, true>(src, gamma, stream_rows, lds, gamma_next, (float*)next, ldn, n_rows, width, eps,
                                               eps_next, stream);
  else
    rl::launch_add_norm_vec<__nv_bfloat16, true, true>(src, gamma, stream_rows, lds, gamma_next, (__nv_bfloat16*)next, ldn, n_rows,
                                                       width, eps, eps_next, stream);
  RL_CHECK_LAUNCH();
  return 0;
}

// stream = rmsnorm(alpha * stream + sigmoid(z + zb) * (s0 * y0 + s1 * y1)) * gamma (y1 may be null; z null: no gate; zb null: no bias), with an optional
// bfloat16 copy of the new rows; see the kernel.
RL_EXPORT int rl_gated_join_norm(const float* y0, long ld0, float s0, const float* y1, long ld1, float s1, const float* z,
                                 long ldz, const float* zb, const float* gamma, float* stream_rows, long lds, void* copy, long ldc,
                                 int n_rows, int width, float eps, float alpha, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (width <= 0 || y0 == nullptr) return -2;
  const int threads = rl::norm_threads(width);
  const size_t row_bytes = (size_t)width * sizeof(float);
  if (row_bytes <= 40 * 1024)
    rl::launch_pdl(rl::gated_join_norm_kernel<true>, n_rows, threads, row_bytes, stream, y0, ld0, s0, y1, ld1, s1, z, ldz,
                   zb, gamma, stream_rows, lds, (__nv_bfloat16*)copy, ldc, n_rows, width, eps, alpha);
  else
    rl::launch_pdl(rl::gated_join_norm_kernel<false>, n_rows, threads, 0, stream, y0, ld0, s0, y1, ld1, s1, z, ldz, zb, gamma,
                   stream_rows, lds, (__nv_bfloat16*)copy, ldc, n_rows, width, eps, alpha);
  RL_CHECK_LAUNCH();
  return 0;
}
