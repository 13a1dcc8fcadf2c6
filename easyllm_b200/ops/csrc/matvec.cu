// y = x · Wᵀ for a few rows of x (decoding) and for row lengths the TMA-fed GEMM cannot take: bound by the weight bytes.
//
// A warp computes NW rows of W against MR rows of x: lanes stride over K with 16-byte loads of W (bf16) and of x (L1),
// fp32 accumulation, one shuffle reduction per result.  KS warps of a CTA may split K when N alone gives too few warps.
// Optional bias, tanh, fp32 output, or accumulation into an fp32 matrix; a batch of equally shaped products in grid.z.
#include "vec.cuh"

namespace ell {

constexpr int kMvWarps = 8;

struct MatvecArgs {
  const void *x, *w, *bias;
  void* out;
  long long xb, wb, ob;       // batch strides in elements
  int M, N, K, ldx, ldo;
  int out_f32, accumulate, act_tanh, ks;
};

template <typename T, int MR, int NW, bool VEC>
__global__ void __launch_bounds__(kMvWarps * 32) matvec_kernel(const MatvecArgs a) {
  __shared__ float red[kMvWarps][NW * MR];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ks = a.ks, part = warp % ks, n0 = (blockIdx.x * (kMvWarps / ks) + warp / ks) * NW, m0 = blockIdx.y * MR;
  const T* x = reinterpret_cast<const T*>(a.x) + blockIdx.z * a.xb + (size_t)m0 * a.ldx;
  const T* w = reinterpret_cast<const T*>(a.w) + blockIdx.z * a.wb + (size_t)n0 * a.K;
  float acc[NW][MR];
#pragma unroll
  for (int i = 0; i < NW; ++i)
#pragma unroll
    for (int m = 0; m < MR; ++m) acc[i][m] = 0.f;
  if (n0 < a.N) {
#pragma unroll 2
    for (int k = (part * 32 + lane) * 8; k < a.K; k += ks * 256) {
      float wf[NW][8];
#pragma unroll
      for (int i = 0; i < NW; ++i) {
        if (VEC && n0 + i < a.N) {
          load_v<8>(w + (size_t)i * a.K + k, wf[i]);
        } else {
#pragma unroll
          for (int j = 0; j < 8; ++j) wf[i][j] = n0 + i < a.N && k + j < a.K ? to_f<T>(w[(size_t)i * a.K + k + j]) : 0.f;
        }
      }
#pragma unroll
      for (int m = 0; m < MR; ++m) {
        float xf[8];
        if (VEC && m0 + m < a.M) {
          load_v<8>(x + (size_t)m * a.ldx + k, xf);
        } else {
#pragma unroll
          for (int j = 0; j < 8; ++j) xf[j] = m0 + m < a.M && k + j < a.K ? to_f<T>(x[(size_t)m * a.ldx + k + j]) : 0.f;
        }
#pragma unroll
        for (int i = 0; i < NW; ++i)
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[i][m] = fmaf(wf[i][j], xf[j], acc[i][m]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NW; ++i)
#pragma unroll
    for (int m = 0; m < MR; ++m) {
      const float v = warp_sum(acc[i][m]);
      if (lane == 0) red[warp][i * MR + m] = v;
    }
  __syncthreads();
  if (part != 0 || n0 >= a.N) return;
  for (int e = lane; e < NW * MR; e += 32) {
    const int i = e / MR, m = e % MR, n = n0 + i;
    if (n >= a.N || m0 + m >= a.M) continue;
    float v = 0.f;
    for (int p = 0; p < ks; ++p) v += red[warp + p][e];
    if (a.bias != nullptr) v += to_f<T>(reinterpret_cast<const T*>(a.bias)[n]);
    if (a.act_tanh) v = tanhf(v);
    const size_t o = blockIdx.z * a.ob + (size_t)(m0 + m) * a.ldo + n;
    if (a.accumulate) reinterpret_cast<float*>(a.out)[o] += v;
    else if (a.out_f32) reinterpret_cast<float*>(a.out)[o] = v;
    else reinterpret_cast<T*>(a.out)[o] = from_f<T>(v);
  }
}

template <typename T, int MR, int NW>
int launch_matvec(MatvecArgs a, int batch, bool vec, cudaStream_t stream) {
  const long long warps = (long long)((a.N + NW - 1) / NW) * ((a.M + MR - 1) / MR) * batch;
  a.ks = 1;
  while (a.ks < kMvWarps && warps * a.ks < 12LL * kNumSMs && a.K >= 512 * a.ks) a.ks *= 2;
  const int per = kMvWarps / a.ks;
  dim3 grid(((a.N + NW - 1) / NW + per - 1) / per, (a.M + MR - 1) / MR, batch);
  if (grid.y > 65535) return -2;
  if (vec) matvec_kernel<T, MR, NW, true><<<grid, kMvWarps * 32, 0, stream>>>(a);
  else matvec_kernel<T, MR, NW, false><<<grid, kMvWarps * 32, 0, stream>>>(a);
  return launch_status();
}

template <typename T>
int dispatch_matvec(const MatvecArgs& a, int batch, bool vec, cudaStream_t stream) {
  if (a.M == 1) return launch_matvec<T, 1, 2>(a, batch, vec, stream);
  if (a.M == 2) return launch_matvec<T, 2, 2>(a, batch, vec, stream);
  if (a.M <= 4) return launch_matvec<T, 4, 2>(a, batch, vec, stream);
  return launch_matvec<T, 8, 4>(a, batch, vec, stream);
}

// ---- mixture of experts: routing, and the per-token products of a few tokens -----------------------
// One warp per token: the `top` largest router logits (ties: the lower index), scores sigmoid(z).
__global__ void moe_route_kernel(const float* __restrict__ z, int* __restrict__ idx, float* __restrict__ w, int n, int E,
                                 int top, int ldz) {
  const int t = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  if (t >= n) return;
  const float* row = z + (size_t)t * ldz;
  uint32_t taken = 0;                                  // bit i: expert 32 i + lane
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int be = 0x7fffffff;
    for (int i = 0; 32 * i + lane < E; ++i)
      if (!(taken >> i & 1)) {
        const float v = row[32 * i + lane];
        if (v > best || be == 0x7fffffff) {
          best = v;
          be = 32 * i + lane;
        }
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (oe != 0x7fffffff && (be == 0x7fffffff || ov > best || (ov == best && oe < be))) {
        best = ov;
        be = oe;
      }
    }
    if ((be & 31) == lane) taken |= 1u << (be >> 5);
    if (lane == 0) {
      idx[t * top + k] = be;
      w[t * top + k] = sigmoid_f(best);
    }
  }
}

// hid[slot][f] = (w_slot relu(up_e[f] . h_token))^2 for slot = token * top + k; a warp computes two hidden units.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) moe_up_kernel(const T* __restrict__ h, const T* __restrict__ up,
                                                     const int* __restrict__ idx, const float* __restrict__ wgt,
                                                     T* __restrict__ hid, int top, int F, int W) {
  const int slot = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int f0 = (blockIdx.x * 8 + warp) * 2;
  if (f0 >= F) return;
  const T* x = h + (size_t)(slot / top) * W;
  const T* u0 = up + ((size_t)idx[slot] * F + f0) * W;
  const bool two = f0 + 1 < F;
  float a0 = 0.f, a1 = 0.f;
#pragma unroll 2
  for (int k = lane * 8; k < W; k += 256) {
    float xf[8], w0[8], w1[8];
    if (VEC) {
      load_v<8>(x + k, xf);
      load_v<8>(u0 + k, w0);
      load_v<8>(u0 + (two ? W : 0) + k, w1);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const bool in = k + j < W;
        xf[j] = in ? to_f<T>(x[k + j]) : 0.f;
        w0[j] = in ? to_f<T>(u0[k + j]) : 0.f;
        w1[j] = in ? to_f<T>(u0[(two ? W : 0) + k + j]) : 0.f;
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      a0 = fmaf(xf[j], w0[j], a0);
      a1 = fmaf(xf[j], w1[j], a1);
    }
  }
  a0 = warp_sum(a0);
  a1 = warp_sum(a1);
  if (lane == 0) {
    const float s = wgt[slot];
    a0 = s * fmaxf(a0, 0.f);
    a1 = s * fmaxf(a1, 0.f);
    hid[(size_t)slot * F + f0] = from_f<T>(a0 * a0);
    if (two) hid[(size_t)slot * F + f0 + 1] = from_f<T>(a1 * a1);
  }
}

// acc[token][n] += sum over the token's experts of down_e[n] . hid; a warp owns two outputs of one token.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) moe_down_kernel(const T* __restrict__ hid, const T* __restrict__ down,
                                                       const int* __restrict__ idx, float* __restrict__ acc, int top, int F,
                                                       int W) {
  const int t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = (blockIdx.x * 8 + warp) * 2;
  if (n0 >= W) return;
  const bool two = n0 + 1 < W;
  float a0 = 0.f, a1 = 0.f;
  for (int s = 0; s < top; ++s) {
    const int slot = t * top + s;
    const T* x = hid + (size_t)slot * F;
    const T* d0 = down + ((size_t)idx[slot] * W + n0) * F;
#pragma unroll 2
    for (int k = lane * 8; k < F; k += 256) {
      float xf[8], w0[8], w1[8];
      if (VEC) {
        load_v<8>(x + k, xf);
        load_v<8>(d0 + k, w0);
        load_v<8>(d0 + (two ? F : 0) + k, w1);
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const bool in = k + j < F;
          xf[j] = in ? to_f<T>(x[k + j]) : 0.f;
          w0[j] = in ? to_f<T>(d0[k + j]) : 0.f;
          w1[j] = in ? to_f<T>(d0[(two ? F : 0) + k + j]) : 0.f;
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        a0 = fmaf(xf[j], w0[j], a0);
        a1 = fmaf(xf[j], w1[j], a1);
      }
    }
  }
  a0 = warp_sum(a0);
  a1 = warp_sum(a1);
  if (lane == 0) {
    acc[(size_t)t * W + n0] += a0;
    if (two) acc[(size_t)t * W + n0 + 1] += a1;
  }
}

// ---- mixture of experts: rows sorted by expert for the grouped GEMM ---------------------------------
// One CTA.  Every expert's rows start at a multiple of 128; tile_expert[i] is the expert of row tile i, *n_tiles their
// number, pos[slot] the row of slot = token * top + k, row_scale[row] its score (rows of the padding: 0).
__global__ void __launch_bounds__(1024) moe_plan_kernel(const int* __restrict__ idx, const float* __restrict__ wgt, int slots,
                                                        int E, int* __restrict__ pos, float* __restrict__ row_scale,
                                                        int* __restrict__ tile_expert, int* __restrict__ n_tiles) {
  __shared__ int count[1024], first[1024], scan[1024];
  const int e = threadIdx.x;
  count[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < slots; i += 1024) atomicAdd(&count[idx[i]], 1);
  __syncthreads();
  const int mine = e < E ? (count[e] + 127) / 128 : 0;
  scan[e] = mine;
  __syncthreads();
  for (int o = 1; o < 1024; o <<= 1) {
    const int v = e >= o ? scan[e - o] : 0;
    __syncthreads();
    scan[e] += v;
    __syncthreads();
  }
  const int t0 = scan[e] - mine;
  first[e] = t0 * 128;
  for (int i = 0; i < mine; ++i) tile_expert[t0 + i] = e;
  for (int i = count[e]; i < mine * 128; ++i) row_scale[t0 * 128 + i] = 0.f;
  if (e == 1023) *n_tiles = scan[1023];
  __syncthreads();
  count[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < slots; i += 1024) {
    const int x = idx[i], r = first[x] + atomicAdd(&count[x], 1);
    pos[i] = r;
    row_scale[r] = wgt[i];
  }
}

// xs[pos[slot]] = h[token], 16 bytes a thread.
__global__ void moe_gather_kernel(const uint4* __restrict__ h, uint4* __restrict__ xs, const int* __restrict__ pos, int slots,
                                  int top, int wv) {
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < (long long)slots * wv;
       i += (long long)gridDim.x * blockDim.x) {
    const int slot = (int)(i / wv), c = (int)(i % wv);
    xs[(size_t)pos[slot] * wv + c] = h[(size_t)(slot / top) * wv + c];
  }
}

// acc[token] += sum over its slots of ys[pos[slot]]
__global__ void moe_combine_kernel(const __nv_bfloat16* __restrict__ ys, const int* __restrict__ pos, float* __restrict__ acc,
                                   int n, int top, int W) {
  const int wv = W / 4;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < (long long)n * wv;
       i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / wv), c = (int)(i % wv) * 4;
    float s[4];
    load_v<4>(acc + (size_t)t * W + c, s);
    for (int k = 0; k < top; ++k) {
      float f[4];
      load_v<4>(ys + (size_t)pos[t * top + k] * W + c, f);
#pragma unroll
      for (int j = 0; j < 4; ++j) s[j] += f[j];
    }
    store_v<4>(acc + (size_t)t * W + c, s);
  }
}

}  // namespace ell

using namespace ell;

// out[b] (M x N, rows of ldo) = x[b] (M x K, rows of ldx) · w[b] (N x K contiguous)^T, `batch` products with the given
// element strides.  out_f32 / accumulate: fp32 output / added to an fp32 output; else the activation type.
ELL_API int ell_matvec(const void* x, const void* w, const void* bias, void* out, long long xb, long long wb, long long ob,
                       int batch, int M, int N, int K, int ldx, int ldo, int out_f32, int accumulate, int act_tanh,
                       int is_bf16, cudaStream_t stream) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  if (batch > 65535) return -2;
  MatvecArgs a{x, w, bias, out, xb, wb, ob, M, N, K, ldx, ldo, out_f32, accumulate, act_tanh, 1};
  const int esz = is_bf16 ? 2 : 4;
  const bool vec = K % 8 == 0 && (ldx * esz) % 16 == 0 && aligned_to(x, 16) && aligned_to(w, 16) && (xb * esz) % 16 == 0 &&
                   (wb * esz) % 16 == 0;
  return is_bf16 ? dispatch_matvec<__nv_bfloat16>(a, batch, vec, stream) : dispatch_matvec<float>(a, batch, vec, stream);
}

ELL_API int ell_moe_route(const float* z, int* idx, float* w, int n, int E, int top, int ldz, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (E > 1024 || top > E || top < 1) return -2;
  moe_route_kernel<<<(n + 7) / 8, 256, 0, stream>>>(z, idx, w, n, E, top, ldz);
  return launch_status();
}

// acc [n, W] fp32 += experts; up [E, F, W], down [E, W, F]; hid: scratch [n * top, F] of the activation type.
ELL_API int ell_moe_rows(const void* h, const void* up, const void* down, const int* idx, const float* w, void* hid,
                         float* acc, int n, int top, int F, int W, int is_bf16, cudaStream_t stream) {
  if (n <= 0) return 0;
  if ((long long)n * top > 65535) return -2;
  const bool v = F % 8 == 0 && W % 8 == 0 && aligned_to(h, 16) && aligned_to(up, 16) && aligned_to(down, 16) && aligned_to(hid, 16);
  dim3 gu((F + 15) / 16, n * top), gd((W + 15) / 16, n);
#define ELL_MOE_ROWS(T, V)                                                                                          \
  moe_up_kernel<T, V><<<gu, 256, 0, stream>>>((const T*)h, (const T*)up, idx, w, (T*)hid, top, F, W);               \
  moe_down_kernel<T, V><<<gd, 256, 0, stream>>>((const T*)hid, (const T*)down, idx, acc, top, F, W);
  if (is_bf16) {
    if (v) { ELL_MOE_ROWS(__nv_bfloat16, true) } else { ELL_MOE_ROWS(__nv_bfloat16, false) }
  } else {
    if (v) { ELL_MOE_ROWS(float, true) } else { ELL_MOE_ROWS(float, false) }
  }
#undef ELL_MOE_ROWS
  return launch_status();
}

// Row plan + gathered rows of the grouped GEMM (bf16, W a multiple of 8).
ELL_API int ell_moe_gather(const void* h, void* xs, const int* idx, const float* w, int* pos, float* row_scale,
                           int* tile_expert, int* n_tiles, int n, int top, int E, int W, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (E > 1024 || W % 8) return -2;
  moe_plan_kernel<<<1, 1024, 0, stream>>>(idx, w, n * top, E, pos, row_scale, tile_expert, n_tiles);
  moe_gather_kernel<<<grid_for((long long)n * top * (W / 8), 256), 256, 0, stream>>>((const uint4*)h, (uint4*)xs, pos,
                                                                                    n * top, top, W / 8);
  return launch_status();
}

ELL_API int ell_moe_combine(const void* ys, const int* pos, float* acc, int n, int top, int W, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (W % 4) return -2;
  moe_combine_kernel<<<grid_for((long long)n * (W / 4), 256), 256, 0, stream>>>((const __nv_bfloat16*)ys, pos, acc, n, top, W);
  return launch_status();
}
