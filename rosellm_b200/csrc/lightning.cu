// Linear attention whose state decays by one fixed factor a head:
//   S_t = d_h S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t,  S [dk, dv] float32 in the request's state slot,
// with q, k, v the (optionally silu'd) columns of one float32 matrix, the packed projections of the layer's input.
// Because d_h does not depend on the token, a portion of n tokens needs no walk over its tokens.  It is cut into
// chunks of 64 (the step's list of 64-token tiles), and with the powers of d_h in a table:
//   `lightning_chunk_*`: what a chunk alone adds to the state, U = sum_j d^(n-1-j) k_j v_j^T, all chunks at once;
//   `lightning_scan_kernel`: the states between the chunks, S <- d^n S + U, a thread an element: leaves in place of
//     each U the state ahead of its chunk, and the portion's last state in the slot;
//   `lightning_out_*`: o_i = d^(i+1) S^T q_i + sum_(j <= i) d^(i-j) (q_i . k_j) v_j, all chunks at once.
// Only non-negative powers occur, so nothing overflows or is divided by whatever the decays are (0 and 1 included).
// Two forms of the first and the last: `_simt` in IEEE float32 multiply-adds (tile_gemm.cuh), and `_mma` on the tensor
// cores, where q, k, v are bfloat16 operands and what is float32 (the decayed scores, the decayed keys, the state) enters
// as the sum of two bfloat16 numbers, so that it loses no more than some 2^-17 of its size; accumulation is float32.
// `lightning_decode_kernel`: a request's single token; the state is read once, updated and written back.
#include "common.cuh"
#include "mma_tile.cuh"
#include "tile_gemm.cuh"

namespace rl {

constexpr int LG_C = 64;  // tokens a chunk

struct LightningParams {
  const float* proj;  // [tokens, ldp]
  long ldp;
  int off_q, off_k, off_v;  // first columns
  const float* powers;      // [heads, LG_C + 1]: powers[h][n] = d_h^n
  float* state;             // [slots, heads, dk, dv], state_stride floats a slot
  long state_stride;
  float* chunks;  // [tiles, heads, dk, dv] scratch
  float* out;     // [tokens, heads * dv]
  const int* q_start;
  const int* slots;
  int n_heads, dk, dv, act;
};

__device__ __forceinline__ float lightning_act(float z, int act) { return act ? z / (1.0f + expf(-z)) : z; }
__device__ __forceinline__ float lightning_act_fast(float z, int act) { return act ? __fdividef(z, 1.0f + __expf(-z)) : z; }

struct LightningTile {
  int req, t0, n, tok;  // request, first of its tokens in this tile, tokens, row of the first in the step
  bool live;
};
__device__ __forceinline__ LightningTile lightning_tile(const LightningParams& p, const int* tiles, int i) {
  LightningTile t;
  t.req = tiles[2 * i];
  t.t0 = tiles[2 * i + 1];
  const int qs = p.q_start[t.req];
  t.n = min(LG_C, p.q_start[t.req + 1] - qs - t.t0);
  t.tok = qs + t.t0;
  t.live = p.slots[t.req] >= 0;  // slot -1: padding of a fixed-size batch
  return t;
}

// ---- float32 --------------------------------------------------------------------------------------------------

// Grid (tiles, heads, pieces of 64 x 64 of the state).
__global__ __launch_bounds__(256) void lightning_chunk_simt_kernel(const LightningParams p, const int* __restrict__ tiles) {
  __shared__ TileGemmSmem s;
  pdl_begin();
  const LightningTile t = lightning_tile(p, tiles, blockIdx.x);
  if (!t.live) return;
  const int h = blockIdx.y, n_pieces = (p.dv + TG_N - 1) / TG_N;
  const int m0 = blockIdx.z / n_pieces * TG_M, n0 = blockIdx.z % n_pieces * TG_N;
  const float* k = p.proj + (size_t)t.tok * p.ldp + p.off_k + h * p.dk + m0;
  const float* v = p.proj + (size_t)t.tok * p.ldp + p.off_v + h * p.dv + n0;
  const float* pw = p.powers + h * (LG_C + 1);
  float acc[4][4] = {};
  tile_gemm(
      acc, t.n,
      [&](int m, int j) { return (j < t.n && m0 + m < p.dk) ? lightning_act(k[(size_t)j * p.ldp + m], p.act) * pw[t.n - 1 - j] : 0.f; },
      [&](int j, int n) { return (j < t.n && n0 + n < p.dv) ? lightning_act(v[(size_t)j * p.ldp + n], p.act) : 0.f; }, s);
  float* u = p.chunks + ((size_t)blockIdx.x * p.n_heads + h) * p.dk * p.dv;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < p.dk && n < p.dv) u[(size_t)m * p.dv + n] = acc[i][j];
    }
}

// Grid (tiles, heads, groups of 64 columns).
__global__ __launch_bounds__(256) void lightning_out_simt_kernel(const LightningParams p, const int* __restrict__ tiles) {
  __shared__ TileGemmSmem s;
  __shared__ float p_s[LG_C][LG_C + 1];
  pdl_begin();
  const LightningTile t = lightning_tile(p, tiles, blockIdx.x);
  const int h = blockIdx.y, n0 = blockIdx.z * TG_N;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const float* q = p.proj + (size_t)t.tok * p.ldp + p.off_q + h * p.dk;
  const float* k = p.proj + (size_t)t.tok * p.ldp + p.off_k + h * p.dk;
  const float* v = p.proj + (size_t)t.tok * p.ldp + p.off_v + h * p.dv + n0;
  const float* pw = p.powers + h * (LG_C + 1);
  const float* st = p.chunks + ((size_t)blockIdx.x * p.n_heads + h) * p.dk * p.dv + n0;
  float acc[4][4] = {}, old[4][4] = {};
  if (t.live) {
    auto query = [&](int m, int c) { return (m < t.n && c < p.dk) ? lightning_act(q[(size_t)m * p.ldp + c], p.act) : 0.f; };
    float sc[4][4] = {};
    tile_gemm(
        sc, p.dk, query,
        [&](int c, int n) { return (n < t.n && c < p.dk) ? lightning_act(k[(size_t)n * p.ldp + c], p.act) : 0.f; }, s);
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int m = ty * 4 + i, n = tx * 4 + j;
        p_s[m][n] = m >= n ? sc[i][j] * pw[m - n] : 0.f;
      }
    __syncthreads();
    tile_gemm(
        acc, t.n, [&](int m, int j) { return p_s[m][j]; },
        [&](int j, int n) { return (j < t.n && n0 + n < p.dv) ? lightning_act(v[(size_t)j * p.ldp + n], p.act) : 0.f; }, s);
    tile_gemm(
        old, p.dk, query, [&](int c, int n) { return (c < p.dk && n0 + n < p.dv) ? st[(size_t)c * p.dv + n] : 0.f; }, s);
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = ty * 4 + i;
    if (m >= t.n) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < p.dv) p.out[(size_t)(t.tok + m) * p.n_heads * p.dv + (size_t)h * p.dv + n] = fmaf(pw[m + 1], old[i][j], acc[i][j]);
    }
  }
}

// ---- the states between the chunks ------------------------------------------------------------------------------

// Grid (requests, heads, pieces of a head's state): a block walks its request's tiles, a thread VEC elements of the state,
// eight chunks' worth fetched at a time.  The tiles lie request by request, so a request's first one is the number of
// tiles of the requests before it (one token: none).
template <int VEC>
__global__ __launch_bounds__(256) void lightning_scan_kernel(const LightningParams p) {
  __shared__ int first_s;
  pdl_begin();
  const int req = blockIdx.x, slot = p.slots[req];
  const int n_tok = p.q_start[req + 1] - p.q_start[req];
  if (slot < 0 || n_tok < 2) return;
  if (threadIdx.x == 0) first_s = 0;
  __syncthreads();
  int before = 0;
  for (int r = threadIdx.x; r < req; r += blockDim.x) {
    const int n = p.q_start[r + 1] - p.q_start[r];
    before += n > 1 ? (n + LG_C - 1) / LG_C : 0;
  }
  if (before) atomicAdd(&first_s, before);
  __syncthreads();
  const int i0 = first_s, h = blockIdx.y, size = p.dk * p.dv;
  const int at = (blockIdx.z * blockDim.x + threadIdx.x) * VEC;
  if (at >= size) return;
  const int n_chunks = (n_tok + LG_C - 1) / LG_C;
  const float* pw = p.powers + h * (LG_C + 1);
  const float d_full = pw[LG_C], d_last = pw[n_tok - (n_chunks - 1) * LG_C];
  float* st = p.state + (size_t)slot * p.state_stride + (size_t)h * size + at;
  float* u = p.chunks + ((size_t)i0 * p.n_heads + h) * size + at;
  const size_t step = (size_t)p.n_heads * size;
  float S[VEC];
  auto get = [&](const float* from, float (&to)[VEC]) {
    if constexpr (VEC == 4) {
      const float4 x = *reinterpret_cast<const float4*>(from);
      to[0] = x.x, to[1] = x.y, to[2] = x.z, to[3] = x.w;
    } else {
      to[0] = *from;
    }
  };
  auto put = [&](float* to, const float (&from)[VEC]) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(to) = make_float4(from[0], from[1], from[2], from[3]);
    else *to = from[0];
  };
  get(st, S);
  constexpr int AHEAD = 8;
  for (int c0 = 0; c0 < n_chunks; c0 += AHEAD) {
    float x[AHEAD][VEC];
#pragma unroll
    for (int a = 0; a < AHEAD; ++a)
      if (c0 + a < n_chunks) get(u + (size_t)(c0 + a) * step, x[a]);
#pragma unroll
    for (int a = 0; a < AHEAD; ++a)
      if (c0 + a < n_chunks) {
        put(u + (size_t)(c0 + a) * step, S);
        const float d = c0 + a == n_chunks - 1 ? d_last : d_full;
#pragma unroll
        for (int e = 0; e < VEC; ++e) S[e] = fmaf(d, S[e], x[a][e]);
      }
  }
  put(st, S);
}

// ---- the tensor cores -------------------------------------------------------------------------------------------

// A block has NG groups of four warps, each group 64 value columns: the queries and keys of a chunk are brought in once
// for all of them.
constexpr int LG_N = 64;
template <int NG>
struct LightningCols {
  static constexpr int N = LG_N * NG, LD = N + 8;  // value columns a block, row of a value or state tile in shared memory
};

__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, const void* row) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"((uint32_t)__cvta_generic_to_shared(row)));
}
__device__ __forceinline__ void mma_kn(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  const uint32_t b[2] = {b0, b1};
  mma_bf16_16x8x16(c, a, b);
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
// `rows` x `cols` elements of a float32 matrix, handed to put(row, column, values) for a tile of `rows_pad` x `cols_pad`, zeros
// outside.  VEC: columns in fours, 16-byte loads.  A thread has eight pieces on their way before it uses the first.
template <bool VEC, class Put>
__device__ __forceinline__ void lightning_stage(const float* src, long ld, int rows, int cols, int rows_pad, int cols_pad, Put put) {
  constexpr int W = VEC ? 4 : 1, BATCH = 8;
  const int per_row = cols_pad / W, dr = blockDim.x / per_row, dc = blockDim.x - dr * per_row;
  int r0 = threadIdx.x / per_row, c0 = threadIdx.x - r0 * per_row;
  auto advance = [&](int& r, int& c) {
    r += dr;
    c += dc;
    if (c >= per_row) {
      c -= per_row;
      ++r;
    }
  };
  while (r0 < rows_pad) {
    float x[BATCH][W];
    int r = r0, c = c0;
#pragma unroll
    for (int b = 0; b < BATCH; ++b) {
      const bool in = r < rows && c * W < cols;
      if constexpr (VEC) {
        const float4 f = in ? *reinterpret_cast<const float4*>(src + (size_t)r * ld + c * W) : make_float4(0.f, 0.f, 0.f, 0.f);
        x[b][0] = f.x, x[b][1] = f.y, x[b][2] = f.z, x[b][3] = f.w;
      } else {
        x[b][0] = in ? src[(size_t)r * ld + c] : 0.f;
      }
      advance(r, c);
    }
#pragma unroll
    for (int b = 0; b < BATCH; ++b) {
      if (r0 < rows_pad) put(r0, c0 * W, x[b]);
      advance(r0, c0);
    }
  }
}
template <int W>
__device__ __forceinline__ void store_bf16(__nv_bfloat16* dst, const float (&x)[W]) {
  if constexpr (W == 4) {
    *reinterpret_cast<uint2*>(dst) = make_uint2(pack2(x[0], x[1]), pack2(x[2], x[3]));
  } else {
    dst[0] = __float2bfloat16_rn(x[0]);
  }
}
// x = hi + lo + (at most 2^-17 |x|)
template <int W>
__device__ __forceinline__ void store_split(__nv_bfloat16* hi, __nv_bfloat16* lo, const float (&x)[W]) {
  float rest[W];
#pragma unroll
  for (int e = 0; e < W; ++e) rest[e] = x[e] - __bfloat162float(__float2bfloat16_rn(x[e]));
  store_bf16(hi, x);
  store_bf16(lo, rest);
}

// Grid (tiles, heads, groups of 64 NG value columns): U of the chunk, rows of 16 keys over a group's four warps in turn.
template <bool VEC, int NG>
__global__ __launch_bounds__(128 * NG) void lightning_chunk_mma_kernel(const LightningParams p, const int* __restrict__ tiles) {
  extern __shared__ __align__(16) unsigned char lightning_smem[];
  __shared__ float pw_s[LG_C + 1];
  using bf16 = __nv_bfloat16;
  constexpr int LDV = LightningCols<NG>::LD, COLS = LightningCols<NG>::N;
  const int h = blockIdx.y, n0 = blockIdx.z * COLS;
  if (threadIdx.x <= LG_C) pw_s[threadIdx.x] = p.powers[h * (LG_C + 1) + threadIdx.x];
  pdl_begin();
  const LightningTile t = lightning_tile(p, tiles, blockIdx.x);
  if (!t.live) return;
  const int dkp = (p.dk + 15) & ~15, LDK = dkp + 8;
  bf16* k_hi = reinterpret_cast<bf16*>(lightning_smem);  // [64][LDK]
  bf16* k_lo = k_hi + LG_C * LDK;
  bf16* v_s = k_lo + LG_C * LDK;  // [64][LDV]
  __syncthreads();
  const float* row = p.proj + (size_t)t.tok * p.ldp;
  lightning_stage<VEC>(row + p.off_k + h * p.dk, p.ldp, t.n, p.dk, LG_C, dkp, [&](int r, int c, auto& x) {
    const float w = r < t.n ? pw_s[t.n - 1 - r] : 0.f;
    for (auto& e : x) e = __bfloat162float(__float2bfloat16_rn(lightning_act_fast(e, p.act))) * w;  // the key as lightning_out_mma_kernel has it
    store_split(k_hi + r * LDK + c, k_lo + r * LDK + c, x);
  });
  lightning_stage<VEC>(row + p.off_v + h * p.dv + n0, p.ldp, t.n, p.dv - n0, LG_C, COLS, [&](int r, int c, auto& x) {
    for (auto& e : x) e = lightning_act_fast(e, p.act);
    store_bf16(v_s + r * LDV + c, x);
  });
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) & 3, g = lane >> 2, q2 = 2 * (lane & 3);
  const int v0 = (threadIdx.x >> 7) * LG_N;  // this group's first column in the tile
  float* u = p.chunks + ((size_t)blockIdx.x * p.n_heads + h) * p.dk * p.dv;
  for (int m0 = warp * 16; m0 < dkp; m0 += 64) {
    float acc[8][4] = {};
#pragma unroll
    for (int j0 = 0; j0 < LG_C; j0 += 16) {
      // A = keys^T: stored token by token, fetched transposed
      uint32_t a_hi[4], a_lo[4];
      const int off = (j0 + (lane & 7) + (lane >> 4) * 8) * LDK + m0 + ((lane >> 3) & 1) * 8;
      ldmatrix_x4_trans(a_hi[0], a_hi[1], a_hi[2], a_hi[3], k_hi + off);
      ldmatrix_x4_trans(a_lo[0], a_lo[1], a_lo[2], a_lo[3], k_lo + off);
#pragma unroll
      for (int nv = 0; nv < 8; nv += 2) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3, v_s + (j0 + (lane & 15)) * LDV + v0 + (nv + (lane >> 4)) * 8);
        mma_kn(acc[nv], a_hi, b0, b1);
        mma_kn(acc[nv + 1], a_hi, b2, b3);
        mma_kn(acc[nv], a_lo, b0, b1);
        mma_kn(acc[nv + 1], a_lo, b2, b3);
      }
    }
#pragma unroll
    for (int nv = 0; nv < 8; ++nv)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int m = m0 + g + half * 8, n = n0 + v0 + nv * 8 + q2;
        if (m >= p.dk || n >= p.dv) continue;
        float* dst = u + (size_t)m * p.dv + n;
        if (VEC) {
          *reinterpret_cast<float2*>(dst) = make_float2(acc[nv][2 * half], acc[nv][2 * half + 1]);
        } else {
          dst[0] = acc[nv][2 * half];
          if (n + 1 < p.dv) dst[1] = acc[nv][2 * half + 1];
        }
      }
  }
}

// Grid (tiles, heads, groups of 64 NG value columns): the chunk's outputs, 16 tokens and 64 columns a warp.
template <bool VEC, int NG>
__global__ __launch_bounds__(128 * NG) void lightning_out_mma_kernel(const LightningParams p, const int* __restrict__ tiles) {
  extern __shared__ __align__(16) unsigned char lightning_smem[];
  __shared__ float pw_s[LG_C + 1];
  using bf16 = __nv_bfloat16;
  constexpr int LDV = LightningCols<NG>::LD, COLS = LightningCols<NG>::N;
  const int h = blockIdx.y, n0 = blockIdx.z * COLS;
  if (threadIdx.x <= LG_C) pw_s[threadIdx.x] = p.powers[h * (LG_C + 1) + threadIdx.x];
  pdl_begin();
  const LightningTile t = lightning_tile(p, tiles, blockIdx.x);
  const int dkp = (p.dk + 15) & ~15, LDK = dkp + 8;
  bf16* q_s = reinterpret_cast<bf16*>(lightning_smem);  // [64][LDK]
  bf16* k_s = q_s + LG_C * LDK;                         // [64][LDK]
  bf16* v_s = k_s + LG_C * LDK;                         // [64][LDV]
  bf16* st_hi = v_s + LG_C * LDV;                    // [dkp][LDV]
  bf16* st_lo = st_hi + dkp * LDV;
  const float* row = p.proj + (size_t)t.tok * p.ldp;
  const int live_rows = t.live ? t.n : 0;
  auto put_act = [&](bf16* dst, int ld) {
    return [=](int r, int c, auto& x) {
      for (auto& e : x) e = lightning_act_fast(e, p.act);
      store_bf16(dst + r * ld + c, x);
    };
  };
  lightning_stage<VEC>(row + p.off_q + h * p.dk, p.ldp, live_rows, p.dk, LG_C, dkp, put_act(q_s, LDK));
  lightning_stage<VEC>(row + p.off_k + h * p.dk, p.ldp, live_rows, p.dk, LG_C, dkp, put_act(k_s, LDK));
  lightning_stage<VEC>(row + p.off_v + h * p.dv + n0, p.ldp, live_rows, p.dv - n0, LG_C, COLS, put_act(v_s, LDV));
  lightning_stage<VEC>(p.chunks + ((size_t)blockIdx.x * p.n_heads + h) * p.dk * p.dv + n0, p.dv, t.live ? p.dk : 0, p.dv - n0, dkp, COLS,
                       [&](int r, int c, auto& x) { store_split(st_hi + r * LDV + c, st_lo + r * LDV + c, x); });
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) & 3, g = lane >> 2, q2 = 2 * (lane & 3);
  const int v0 = (threadIdx.x >> 7) * LG_N;  // this group's first column in the tile
  if (warp * 16 >= t.n) return;
  const int row_a = warp * 16 + g, row_b = row_a + 8;  // tokens of the chunk
  const int key_tiles = 2 * (warp + 1);                // tiles of eight keys up to the warp's last token
  float sc[8][4] = {}, o[8][4] = {};
  for (int c0 = 0; c0 < dkp; c0 += 16) {
    uint32_t a[4];
    ldmatrix_x4(a[0], a[1], a[2], a[3], q_s + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDK + c0 + (lane >> 4) * 8);
#pragma unroll
    for (int nk = 0; nk < 8; nk += 2) {
      if (nk < key_tiles) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(b0, b1, b2, b3, k_s + (nk * 8 + (lane & 7) + (lane >> 4) * 8) * LDK + c0 + ((lane >> 3) & 1) * 8);
        mma_kn(sc[nk], a, b0, b1);
        mma_kn(sc[nk + 1], a, b2, b3);
      }
    }
#pragma unroll
    for (int nv = 0; nv < 8; nv += 2) {
      uint32_t b0, b1, b2, b3;
      const int off = (c0 + (lane & 15)) * LDV + v0 + (nv + (lane >> 4)) * 8;
      ldmatrix_x4_trans(b0, b1, b2, b3, st_hi + off);
      mma_kn(o[nv], a, b0, b1);
      mma_kn(o[nv + 1], a, b2, b3);
      ldmatrix_x4_trans(b0, b1, b2, b3, st_lo + off);
      mma_kn(o[nv], a, b0, b1);
      mma_kn(o[nv + 1], a, b2, b3);
    }
  }
  const float d_a = pw_s[row_a + 1], d_b = pw_s[row_b + 1];
#pragma unroll
  for (int nv = 0; nv < 8; ++nv) {
    o[nv][0] *= d_a; o[nv][1] *= d_a; o[nv][2] *= d_b; o[nv][3] *= d_b;
  }
  // the decayed scores, repacked from the accumulators' layout into A fragments of 16 keys
#pragma unroll
  for (int nk = 0; nk < 8; nk += 2) {
    if (nk < key_tiles) {
      uint32_t a_hi[4], a_lo[4];
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = half ? row_b : row_a, j = (nk + x) * 8 + q2;
          const float p0 = i >= j ? sc[nk + x][2 * half] * pw_s[i - j] : 0.f;
          const float p1 = i >= j + 1 ? sc[nk + x][2 * half + 1] * pw_s[i - j - 1] : 0.f;
          const float h0 = __bfloat162float(__float2bfloat16_rn(p0)), h1 = __bfloat162float(__float2bfloat16_rn(p1));
          a_hi[2 * x + half] = pack2(h0, h1);
          a_lo[2 * x + half] = pack2(p0 - h0, p1 - h1);
        }
#pragma unroll
      for (int nv = 0; nv < 8; nv += 2) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3, v_s + (nk * 8 + (lane & 15)) * LDV + v0 + (nv + (lane >> 4)) * 8);
        mma_kn(o[nv], a_hi, b0, b1);
        mma_kn(o[nv + 1], a_hi, b2, b3);
        mma_kn(o[nv], a_lo, b0, b1);
        mma_kn(o[nv + 1], a_lo, b2, b3);
      }
    }
  }
#pragma unroll
  for (int nv = 0; nv < 8; ++nv)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = half ? row_b : row_a, n = n0 + v0 + nv * 8 + q2;
      if (i >= t.n || n >= p.dv) continue;
      float* dst = p.out + (size_t)(t.tok + i) * p.n_heads * p.dv + (size_t)h * p.dv + n;
      if (VEC) {
        *reinterpret_cast<float2*>(dst) = make_float2(o[nv][2 * half], o[nv][2 * half + 1]);
      } else {
        dst[0] = o[nv][2 * half];
        if (n + 1 < p.dv) dst[1] = o[nv][2 * half + 1];
      }
    }
}

// ---- a request's single token -----------------------------------------------------------------------------------

// Grid (decoded requests, heads, groups of `cv` column vectors of VEC).  Thread (row group, column vector): the
// threads of a row group lie side by side along the state's rows.  The state's rows that a thread takes first are on
// their way before the wait for the projections: they were last written in an earlier step, and a copy to the device
// lies between steps.
template <int VEC>
__global__ __launch_bounds__(256) void lightning_decode_kernel(const LightningParams p, const int* __restrict__ decode_reqs, int cv) {
  extern __shared__ float decode_s[];  // q [dk], k [dk], then [row groups][cv * VEC]
  constexpr int AHEAD = 8;
  const int req = decode_reqs[blockIdx.x], h = blockIdx.y;
  const int slot = p.slots[req], tok = p.q_start[req];
  const int groups = blockDim.x / cv, rg = threadIdx.x / cv, c = threadIdx.x - rg * cv;
  const int col = (blockIdx.z * cv + c) * VEC;
  const bool works = slot >= 0 && rg < groups && col < p.dv;
  float* st = p.state + (size_t)(slot < 0 ? 0 : slot) * p.state_stride + (size_t)h * p.dk * p.dv + col;
  auto get = [&](int r, float (&to)[VEC]) {
    if constexpr (VEC == 4) {
      const float4 x = *reinterpret_cast<const float4*>(st + (size_t)r * p.dv);
      to[0] = x.x, to[1] = x.y, to[2] = x.z, to[3] = x.w;
    } else {
      to[0] = st[(size_t)r * p.dv];
    }
  };
  float S[AHEAD][VEC];
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  if (works)
#pragma unroll
    for (int a = 0; a < AHEAD; ++a)
      if (rg + a * groups < p.dk) get(rg + a * groups, S[a]);
  const float d = p.powers[h * (LG_C + 1) + 1];
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const float* row = p.proj + (size_t)tok * p.ldp;
  float* q_s = decode_s;
  float* k_s = q_s + p.dk;
  float* sum_s = k_s + p.dk;
  for (int i = threadIdx.x; i < p.dk; i += blockDim.x) {
    q_s[i] = lightning_act(row[p.off_q + h * p.dk + i], p.act);
    k_s[i] = lightning_act(row[p.off_k + h * p.dk + i], p.act);
  }
  float v[VEC] = {}, o[VEC] = {};
  if (works)
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = lightning_act(row[p.off_v + h * p.dv + col + e], p.act);
  __syncthreads();
  if (works) {
    for (int r0 = rg; r0 < p.dk; r0 += AHEAD * groups) {
      if (r0 != rg)
#pragma unroll
        for (int a = 0; a < AHEAD; ++a)
          if (r0 + a * groups < p.dk) get(r0 + a * groups, S[a]);
#pragma unroll
      for (int a = 0; a < AHEAD; ++a) {
        const int r = r0 + a * groups;
        if (r >= p.dk) continue;
        const float kr = k_s[r], qr = q_s[r];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          S[a][e] = fmaf(d, S[a][e], kr * v[e]);
          o[e] = fmaf(qr, S[a][e], o[e]);
        }
        if constexpr (VEC == 4)
          *reinterpret_cast<float4*>(st + (size_t)r * p.dv) = make_float4(S[a][0], S[a][1], S[a][2], S[a][3]);
        else
          st[(size_t)r * p.dv] = S[a][0];
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) sum_s[(rg * cv + c) * VEC + e] = o[e];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < cv * VEC; i += blockDim.x) {
    const int at = blockIdx.z * cv * VEC + i;
    if (at >= p.dv) continue;
    float total = 0.f;
    if (slot >= 0)
      for (int x = 0; x < groups; ++x) total += sum_s[x * cv * VEC + i];
    p.out[(size_t)tok * p.n_heads * p.dv + (size_t)h * p.dv + at] = total;
  }
}

// ---- the merged heads' norm and gate ----------------------------------------------------------------------------

// out[i] = x[i] / sqrt(mean(x[i]^2) + eps) * gamma * sigmoid(gate[i]), a block a row; gate float32, rows ldg apart.
template <typename TOut, bool VEC>
__global__ __launch_bounds__(256) void rmsnorm_gate_kernel(const float* __restrict__ x, long ldx, const float* __restrict__ gate,
                                                           long ldg, const float* __restrict__ gamma, TOut* __restrict__ out,
                                                           long ldo, int n_rows, int width, float eps) {
  __shared__ float scratch[33];
  pdl_begin();
  const int i = blockIdx.x;
  if (i >= n_rows) return;
  const float* xr = x + (size_t)i * ldx;
  const float* gr = gate + (size_t)i * ldg;
  TOut* o = out + (size_t)i * ldo;
  constexpr int W = VEC ? 4 : 1, KEEP = 4;  // a thread's first pieces stay in registers between the two passes
  const int pieces = width / W;
  float keep[KEEP][W], s = 0.f;
  auto get = [&](const float* from, int d, float (&to)[W]) {
    if constexpr (VEC) {
      const float4 f = reinterpret_cast<const float4*>(from)[d];
      to[0] = f.x, to[1] = f.y, to[2] = f.z, to[3] = f.w;
    } else {
      to[0] = from[d];
    }
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int d = threadIdx.x + k * blockDim.x;
    if (d < pieces) {
      get(xr, d, keep[k]);
#pragma unroll
      for (int e = 0; e < W; ++e) s = fmaf(keep[k][e], keep[k][e], s);
    }
  }
  for (int d = threadIdx.x + KEEP * blockDim.x; d < pieces; d += blockDim.x) {
    float v[W];
    get(xr, d, v);
#pragma unroll
    for (int e = 0; e < W; ++e) s = fmaf(v[e], v[e], s);
  }
  const float r = 1.0f / sqrtf(block_sum(s, scratch) / (float)width + eps);
  auto finish = [&](int d, const float (&v)[W]) {
    float g[W], w[W];
    get(gr, d, g);
    get(gamma, d, w);
#pragma unroll
    for (int e = 0; e < W; ++e) g[e] = v[e] * r * w[e] / (1.0f + expf(-g[e]));
    if constexpr (VEC && sizeof(TOut) == 2) {
      reinterpret_cast<uint2*>(o)[d] = make_uint2(pack2(g[0], g[1]), pack2(g[2], g[3]));
    } else if constexpr (VEC) {
      reinterpret_cast<float4*>(o)[d] = make_float4(g[0], g[1], g[2], g[3]);
    } else {
      o[d] = from_f32<TOut>(g[0]);
    }
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int d = threadIdx.x + k * blockDim.x;
    if (d < pieces) finish(d, keep[k]);
  }
  for (int d = threadIdx.x + KEEP * blockDim.x; d < pieces; d += blockDim.x) {
    float v[W];
    get(xr, d, v);
    finish(d, v);
  }
}

static int lightning_sms() {
  static int sms = 0;
  if (sms == 0) {
    int dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    if (sms <= 0) sms = 148;
  }
  return sms;
}

template <class Kernel>
static void lightning_mma_launch(Kernel kernel, bool& ready, dim3 grid, size_t smem, cudaStream_t stream, const LightningParams& p,
                                 const int* tiles, int groups) {
  if (!ready) {
    note_launch(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    note_launch(cudaFuncSetAttribute(kernel, cudaFuncAttributePreferredSharedMemoryCarveout, (int)cudaSharedmemCarveoutMaxShared));
    ready = true;
  }
  launch_pdl_split(false, kernel, grid, dim3(128 * groups), smem, stream, p, tiles);
}

template <bool VEC, int NG, class Scan>
static void lightning_mma_form(const LightningParams& p, const int* tiles, int n_tiles, cudaStream_t stream, Scan scan) {
  static bool ready[2] = {false, false};
  const int dkp = (p.dk + 15) & ~15, ldk = dkp + 8, ldv = LightningCols<NG>::LD;
  const dim3 grid(n_tiles, p.n_heads, (p.dv + LightningCols<NG>::N - 1) / LightningCols<NG>::N);
  lightning_mma_launch(lightning_chunk_mma_kernel<VEC, NG>, ready[0], grid, (size_t)(2 * LG_C * ldk + LG_C * ldv) * 2, stream, p, tiles, NG);
  scan();
  lightning_mma_launch(lightning_out_mma_kernel<VEC, NG>, ready[1], grid, (size_t)(2 * LG_C * ldk + (LG_C + 2 * dkp) * ldv) * 2, stream, p,
                       tiles, NG);
}
template <class Scan>
static void lightning_mma(bool vec, bool wide, const LightningParams& p, const int* tiles, int n_tiles, cudaStream_t stream, Scan scan) {
  if (vec && wide) lightning_mma_form<true, 2>(p, tiles, n_tiles, stream, scan);
  else if (vec) lightning_mma_form<true, 1>(p, tiles, n_tiles, stream, scan);
  else if (wide) lightning_mma_form<false, 2>(p, tiles, n_tiles, stream, scan);
  else lightning_mma_form<false, 1>(p, tiles, n_tiles, stream, scan);
}

}  // namespace rl

// One step for every request of the step.  proj float32 [tokens, ldp] with the queries, keys (heads * dk columns each)
// and values (heads * dv) from the given columns on; act: 1 for silu on all three, 0 for none; powers float32 [heads,
// 65], powers[h][n] = d_h^n; state float32, state_stride floats a slot; tiles [n_tiles][2]: (request, first token) of the
// 64-token tiles of all requests with more than one token, in the requests' and the tokens' order; decode_reqs: requests with one token; chunks: float32
// scratch [n_tiles, heads, dk, dv]; out float32 [tokens, heads * dv].  tensor_cores: portions on the bfloat16 operands.
RL_EXPORT int rl_lightning(const float* proj, long ldp, int off_q, int off_k, int off_v, int act, const float* powers,
                           float* state, long state_stride, const int* q_start, const int* slots, int n_reqs, const int* tiles, int n_tiles,
                           const int* decode_reqs, int n_decode, float* chunks, float* out, int n_heads, int dk, int dv,
                           int tensor_cores, cudaStream_t stream) {
  if (n_heads <= 0 || n_heads > 65535 || dk <= 0 || dk > 256 || dv <= 0 || dv > 256 || n_tiles < 0 || n_decode < 0 || n_reqs < 0 ||
      state_stride < (long)n_heads * dk * dv || (n_tiles > 0 && chunks == nullptr))
    return -2;
  const rl::LightningParams p{proj, ldp, off_q, off_k, off_v, powers, state, state_stride, chunks, out, q_start, slots,
                              n_heads, dk, dv, act};
  const bool state4 = dv % 4 == 0 && state_stride % 4 == 0 && (uintptr_t)state % 16 == 0;
  if (n_tiles > 0) {
    const int groups = (dv + 63) / 64;
    const dim3 out_grid(n_tiles, n_heads, groups);
    auto scan = [&] {
      rl::launch_pdl(state4 ? rl::lightning_scan_kernel<4> : rl::lightning_scan_kernel<1>,
                     dim3(n_reqs, n_heads, (dk * dv / (state4 ? 4 : 1) + 255) / 256), 256, 0, stream, p);
    };
    if (tensor_cores) {
      const bool vec = state4 && dk % 4 == 0 && ldp % 4 == 0 && off_q % 4 == 0 && off_k % 4 == 0 && off_v % 4 == 0 &&
                       (uintptr_t)proj % 16 == 0 && (uintptr_t)chunks % 16 == 0 && (uintptr_t)out % 16 == 0;
      const bool wide = dv > 64 && dk <= 128;  // two groups of columns a block, where its shared memory has room for their states
      rl::lightning_mma(vec, wide, p, tiles, n_tiles, stream, scan);
    } else {
      rl::launch_pdl(rl::lightning_chunk_simt_kernel, dim3(n_tiles, n_heads, (dk + 63) / 64 * groups), 256, 0, stream, p, tiles);
      scan();
      rl::launch_pdl(rl::lightning_out_simt_kernel, out_grid, 256, 0, stream, p, tiles);
    }
  }
  if (n_decode > 0) {
    const int vecs = state4 ? dv / 4 : dv;
    // column vectors a block: all of a row up to 32, halved (down to 8: 128 bytes of a row) until the grid fills the SMs
    int cv = vecs < 32 ? vecs : 32;
    while (cv >= 16 && (long)n_decode * n_heads * ((vecs + cv - 1) / cv) < rl::lightning_sms()) cv = (cv + 1) / 2;
    const size_t smem = ((size_t)2 * dk + (size_t)(256 / cv) * cv * (state4 ? 4 : 1)) * sizeof(float);
    rl::launch_pdl(state4 ? rl::lightning_decode_kernel<4> : rl::lightning_decode_kernel<1>,
                   dim3(n_decode, n_heads, (vecs + cv - 1) / cv), 256, smem, stream, p, decode_reqs, cv);
  }
  RL_CHECK_LAUNCH();
  return 0;
}

// out = x / sqrt(mean(x^2) + eps) * gamma * sigmoid(gate), row by row.  out_dtype: RL_F32 or RL_BF16.
RL_EXPORT int rl_rmsnorm_gate(int out_dtype, const float* x, long ldx, const float* gate, long ldg, const float* gamma, void* out,
                              long ldo, int n_rows, int width, float eps, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (width <= 0) return -2;
  const int esize = out_dtype == RL_F32 ? 4 : 2;
  const bool vec = width % 4 == 0 && ldx % 4 == 0 && ldg % 4 == 0 && ldo % 4 == 0 && (uintptr_t)x % 16 == 0 &&
                   (uintptr_t)gate % 16 == 0 && (uintptr_t)gamma % 16 == 0 && (uintptr_t)out % (4 * esize) == 0;
  int threads = ((vec ? width / 4 : width) + 31) / 32 * 32;
  threads = threads > 256 ? 256 : threads;
  if (out_dtype == RL_F32)
    rl::launch_pdl(vec ? rl::rmsnorm_gate_kernel<float, true> : rl::rmsnorm_gate_kernel<float, false>, n_rows, threads, 0, stream, x,
                   ldx, gate, ldg, gamma, (float*)out, ldo, n_rows, width, eps);
  else
    rl::launch_pdl(vec ? rl::rmsnorm_gate_kernel<__nv_bfloat16, true> : rl::rmsnorm_gate_kernel<__nv_bfloat16, false>, n_rows, threads,
                   0, stream, x, ldx, gate, ldg, gamma, (__nv_bfloat16*)out, ldo, n_rows, width, eps);
  RL_CHECK_LAUNCH();
  return 0;
}
