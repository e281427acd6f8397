// A residual stream kept in several copies (hyper-connections), float32 throughout:
//
//   a sublayer reads    u = sum_s a_s X_s            (a: one weight a copy)
//   and writes          X'_t = sum_s M[s, t] X_s + b_t y, every t from the old copies   (M indexed [from, to])
//
// `hyper_step_kernel` is everything between two sublayers in one pass over a token's copies (fused: the write of the
// sublayer that has ended, the read of the one that follows, and the RMS norm ahead of it):
//   WRITE: X' as above from X and y.  X may be one row for all copies (stream stride 0): the embedding's output before
//          the first write, which then spreads it.
//   READ:  h = norm(sum_s a_s X'_s) * gamma in the activation type.
//   else:  the copies' sum, what is left of them when nothing reads them any more.
// y is a float32 row a token, or the experts' outputs still lying by place (fused: the weighted sum at the
// end of a mixture of experts): y = sum_j w[t, j] eo[place[t, j]] + sigmoid(sg[t]) shared[t], as `moe_combine_kernel`
// would form it.
// A block a token; a thread's columns of all copies in registers; the row u in shared memory between the statistic
// and the scaling.
#include "common.cuh"

namespace rl {

struct HyperStepParams {
  const float* x;  // [tokens][copies][width]: token stride ldx, copy stride x_copy (0: one row for all copies)
  long ldx, x_copy;
  float* x_new;    // the copies after the write: token stride ldn, copy stride width; or null (not kept)
  long ldn;
  const float* y;  // [tokens, width] (row stride ldy); null with the experts' outputs
  long ldy;
  const float *mix, *out_w;  // WRITE: [copies][copies] from, to; [copies]
  const float* in_w;         // READ: [copies]
  const float* gamma;
  float eps;
  void* h;     // READ: [tokens, width] (row stride ldh)
  long ldh;
  float* sum;  // not READ: [tokens, width] (row stride lds)
  long lds;
  int n_tokens, copies, width;
  // the experts' outputs (eo null: y is given)
  const float* eo;       // [places, width]
  const float* weights;  // [tokens, top] or null (1)
  const int* place_of;   // [tokens, top]
  int top;
  const float* shared;   // [tokens, width] (row stride ld_shared) or null
  long ld_shared;
  const float* sg;       // logits, one a token, stride ldsg; null: a factor of 1
  long ldsg;
};

// V columns at a time: 4 (16-byte accesses) or 1.
template <int V>
struct HyperVec {
  float v[V];
  __device__ __forceinline__ void load(const float* p) {
    if constexpr (V == 4) {
      const float4 t = *reinterpret_cast<const float4*>(p);
      v[0] = t.x, v[1] = t.y, v[2] = t.z, v[3] = t.w;
    } else {
      v[0] = *p;
    }
  }
  __device__ __forceinline__ void store(float* p) const {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
  }
};

// S: the copies, at most (registers); p.copies of them are there.
template <typename TOut, int S, int V, bool WRITE, bool READ>
__global__ __launch_bounds__(256) void hyper_step_kernel(const HyperStepParams p) {
  extern __shared__ __align__(16) float u_s[];  // READ: [width]
  __shared__ float scratch[33];
  __shared__ float coef[S * S + 2 * S];
  pdl_begin();
  const int t = blockIdx.x;
  if (t >= p.n_tokens) return;
  const int n = p.copies;
  float* mix = coef;             // [from][to], row length S
  float* out_w = coef + S * S;
  float* in_w = out_w + S;
  for (int i = threadIdx.x; i < S * S + 2 * S; i += blockDim.x) {
    float c = 0.f;  // copies beyond p.copies count as zero
    if (i < S * S) {
      if (WRITE && i / S < n && i % S < n) c = p.mix[(i / S) * n + i % S];
    } else if (i < S * S + S) {
      if (WRITE && i - S * S < n) c = p.out_w[i - S * S];
    } else if (READ && i - S * S - S < n) {
      c = p.in_w[i - S * S - S];
    }
    coef[i] = c;
  }
  __syncthreads();
  const float* xr = p.x + (size_t)t * p.ldx;
  float gate = 1.f;
  if (WRITE && p.eo != nullptr && p.shared != nullptr && p.sg != nullptr) gate = 1.0f / (1.0f + expf(-p.sg[(size_t)t * p.ldsg]));
  float ss = 0.f;
  for (int d = threadIdx.x * V; d < p.width; d += blockDim.x * V) {
    HyperVec<V> x[S], r[S], y;
#pragma unroll
    for (int s = 0; s < S; ++s) {
      if (s < n) {
        if (s == 0 || p.x_copy != 0) x[s].load(xr + s * p.x_copy + d);
        else x[s] = x[0];
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) x[s].v[e] = 0.f;
      }
    }
    if constexpr (WRITE) {
      if (p.eo == nullptr) {
        y.load(p.y + (size_t)t * p.ldy + d);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) y.v[e] = 0.f;
        for (int j = 0; j < p.top; ++j) {
          HyperVec<V> o;
          o.load(p.eo + (size_t)p.place_of[(size_t)t * p.top + j] * p.width + d);
          const float w = p.weights != nullptr ? p.weights[(size_t)t * p.top + j] : 1.0f;
#pragma unroll
          for (int e = 0; e < V; ++e) y.v[e] = fmaf(w, o.v[e], y.v[e]);
        }
        if (p.shared != nullptr) {
          HyperVec<V> o;
          o.load(p.shared + (size_t)t * p.ld_shared + d);
#pragma unroll
          for (int e = 0; e < V; ++e) y.v[e] = fmaf(gate, o.v[e], y.v[e]);
        }
      }
#pragma unroll
      for (int to = 0; to < S; ++to) {
#pragma unroll
        for (int e = 0; e < V; ++e) {
          float a = 0.f;
#pragma unroll
          for (int s = 0; s < S; ++s) a = fmaf(mix[s * S + to], x[s].v[e], a);
          r[to].v[e] = fmaf(out_w[to], y.v[e], a);
        }
        if (to < n && p.x_new != nullptr) r[to].store(p.x_new + (size_t)t * p.ldn + (size_t)to * p.width + d);
      }
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) r[s] = x[s];
    }
    HyperVec<V> u;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      float a = 0.f;
#pragma unroll
      for (int s = 0; s < S; ++s) a = READ ? fmaf(in_w[s], r[s].v[e], a) : a + r[s].v[e];
      u.v[e] = a;
      ss = fmaf(a, a, ss);
    }
    u.store(READ ? u_s + d : p.sum + (size_t)t * p.lds + d);
  }
  if constexpr (READ) {
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)p.width + p.eps);
    TOut* h = reinterpret_cast<TOut*>(p.h) + (size_t)t * p.ldh;
    for (int d = threadIdx.x * V; d < p.width; d += blockDim.x * V) {  // a thread meets the entries it wrote itself
      HyperVec<V> u, g;
      u.load(u_s + d);
      g.load(p.gamma + d);
#pragma unroll
      for (int e = 0; e < V; ++e) u.v[e] = u.v[e] * inv * g.v[e];
      if constexpr (V == 4 && sizeof(TOut) == 2) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(u.v[0], u.v[1]), hi = __floats2bfloat162_rn(u.v[2], u.v[3]);
        *reinterpret_cast<uint2*>(h + d) =
            make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) h[d + e] = from_f32<TOut>(u.v[e]);
      }
    }
  }
}

template <typename TOut, int S, int V>
static void launch_hyper(const HyperStepParams& p, bool write, bool read, cudaStream_t stream) {
  const size_t smem = read ? (size_t)p.width * sizeof(float) : 0;
  int threads = ((p.width + V - 1) / V + 31) / 32 * 32;
  threads = threads > 256 ? 256 : threads;
  if (write && read) launch_pdl(hyper_step_kernel<TOut, S, V, true, true>, p.n_tokens, threads, smem, stream, p);
  else if (write) launch_pdl(hyper_step_kernel<TOut, S, V, true, false>, p.n_tokens, threads, smem, stream, p);
  else launch_pdl(hyper_step_kernel<TOut, S, V, false, true>, p.n_tokens, threads, smem, stream, p);
}

template <typename TOut, int V>
static void dispatch_hyper(const HyperStepParams& p, bool write, bool read, cudaStream_t stream) {
  if (p.copies == 1) launch_hyper<TOut, 1, V>(p, write, read, stream);
  else if (p.copies == 2) launch_hyper<TOut, 2, V>(p, write, read, stream);
  else if (p.copies == 3) launch_hyper<TOut, 3, V>(p, write, read, stream);
  else if (p.copies == 4) launch_hyper<TOut, 4, V>(p, write, read, stream);
  else if (p.copies <= 8) launch_hyper<TOut, 8, V>(p, write, read, stream);
  else launch_hyper<TOut, 16, 1>(p, write, read, stream);
}

}  // namespace rl

// The step between two sublayers; see the kernel.  copies: 1 to 16; width at most 12,000 where something is read
// (-3 beyond).  mix null: nothing is written (a first read); gamma null: nothing is read, `sum` receives the copies' sum.
// h_dtype: RL_F32 or RL_BF16.
RL_EXPORT int rl_hyper_step(int h_dtype, const float* x, long ldx, long x_copy, float* x_new, long ldn, const float* y, long ldy,
                            const float* mix, const float* out_w, const float* in_w, const float* gamma, float eps, void* h,
                            long ldh, float* sum, long lds, int n_tokens, int copies, int width, const float* eo,
                            const float* weights, const int* place_of, int top, const float* shared, long ld_shared,
                            const float* sg, long ldsg, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  const bool write = mix != nullptr, read = gamma != nullptr;
  if (copies < 1 || copies > 16 || width <= 0 || (!write && !read) || (write && out_w == nullptr) ||
      (write && y == nullptr && (eo == nullptr || place_of == nullptr || top <= 0)) || (read && (in_w == nullptr || h == nullptr)) ||
      (!read && sum == nullptr) || (shared == nullptr && sg != nullptr))
    return -2;
  if (read && width > 12000) return -3;
  const rl::HyperStepParams p{x, ldx, x_copy, x_new, ldn, y, ldy, mix, out_w, in_w, gamma, eps, h, ldh, sum, lds, n_tokens,
                              copies, width, y != nullptr ? nullptr : eo, weights, place_of, top, shared, ld_shared, sg, ldsg};
  const uintptr_t at = (uintptr_t)x | (uintptr_t)x_new | (uintptr_t)y | (uintptr_t)gamma | (uintptr_t)h | (uintptr_t)sum |
                       (uintptr_t)p.eo | (uintptr_t)shared;
  const bool vec = ((width | ldx | x_copy | ldn | ldy | ldh | lds | ld_shared) & 3) == 0 && (at & 15) == 0;
  if (h_dtype == RL_F32) {
    if (vec) rl::dispatch_hyper<float, 4>(p, write, read, stream);
    else rl::dispatch_hyper<float, 1>(p, write, read, stream);
  } else {
    if (vec) rl::dispatch_hyper<__nv_bfloat16, 4>(p, write, read, stream);
    else rl::dispatch_hyper<__nv_bfloat16, 1>(p, write, read, stream);
  }
  RL_CHECK_LAUNCH();
  return 0;
}
