// Logits bounded smoothly: z <- cap * tanh(z / cap), in place, float32.  Where the head's product chooses the tokens
// itself the same function sits in its epilogue (SampleArgs::soft_cap), so a step that samples there launches nothing here.
#include "gemm_epilogue.cuh"

namespace rl {

template <bool VEC>
__global__ __launch_bounds__(256) void soft_cap_kernel(float* __restrict__ z, long n, float cap) {
  pdl_begin();
  const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  if (VEC) {
    float4 v = reinterpret_cast<float4*>(z)[i];
    v.x = soft_capped(v.x, cap);
    v.y = soft_capped(v.y, cap);
    v.z = soft_capped(v.z, cap);
    v.w = soft_capped(v.w, cap);
    reinterpret_cast<float4*>(z)[i] = v;
  } else {
    z[i] = soft_capped(z[i], cap);
  }
}

}  // namespace rl

// n contiguous elements; cap > 0.
RL_EXPORT int rl_soft_cap(float* z, long n, float cap, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (!(cap > 0.f)) return -2;
  const bool vec = n % 4 == 0 && (uintptr_t)z % 16 == 0;
  const long units = vec ? n / 4 : n;
  if ((units + 255) / 256 > 0x7fffffffL) return -2;
  rl::launch_pdl(vec ? rl::soft_cap_kernel<true> : rl::soft_cap_kernel<false>, (unsigned)((units + 255) / 256), 256, 0, stream, z,
                 units, cap);
  RL_CHECK_LAUNCH();
  return 0;
}
