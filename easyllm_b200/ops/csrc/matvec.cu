// y = x · Wᵀ for a few rows of x (decoding) and for row lengths the TMA-fed GEMM cannot take: bound by the weight bytes.
//
// bf16: a warp multiplies 16 rows of W with up to 16 rows of x on mma.sync m16n8k16 (the products are few, the point is
// to keep the instruction count far below the load rate): a thread loads 8 consecutive k of a row with one 16-byte load
// and feeds them to two instructions, in an order of k that is the same for both operands.  The warps of a CTA split K.
// fp32, and shapes without 16-byte rows: a warp computes NW rows of W against MR rows of x, lanes striding over K, fp32
// fused multiply-adds, one shuffle reduction per result.
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

__device__ __forceinline__ void mma_16816(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// MT tiles of 8 rows of x (from row blockIdx.y * 8 MT on).  Rows of W and of x past the end are clamped (their results are dropped); k past the end is
// clamped too, with x taken as zero.
template <int MT>
__global__ void __launch_bounds__(kMvWarps * 32) matvec_mma_kernel(const MatvecArgs a) {
  __shared__ float red[kMvWarps][16][8 * MT + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int ks = a.ks, part = warp % ks, n0 = (blockIdx.x * (kMvWarps / ks) + warp / ks) * 16;
  const int m0 = blockIdx.y * 8 * MT, M = a.M - m0;
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(a.x) + blockIdx.z * a.xb + (size_t)m0 * a.ldx;
  const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(a.w) + blockIdx.z * a.wb;
  const __nv_bfloat16* w0 = w + (size_t)min(n0 + g, a.N - 1) * a.K;
  const __nv_bfloat16* w1 = w + (size_t)min(n0 + g + 8, a.N - 1) * a.K;
  const __nv_bfloat16* xr[MT];
#pragma unroll
  for (int m = 0; m < MT; ++m) xr[m] = x + (size_t)min(m * 8 + g, M - 1) * a.ldx;
  float c0[MT][4], c1[MT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 4; ++i) c0[m][i] = c1[m][i] = 0.f;
  constexpr int U = 4;
  const int nkb = (a.K + 31) / 32;
  for (int kb = part; kb < nkb; kb += ks * U) {
    uint4 wa[U], wb[U], xv[U][MT];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = (kb + u * ks) * 32 + t * 8;
      const bool in = k < a.K;
      const int kc = in ? k : 0;
      wa[u] = *reinterpret_cast<const uint4*>(w0 + kc);
      wb[u] = *reinterpret_cast<const uint4*>(w1 + kc);
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        xv[u][m] = *reinterpret_cast<const uint4*>(xr[m] + kc);
        if (!in) xv[u][m] = make_uint4(0, 0, 0, 0);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        mma_16816(c0[m], wa[u].x, wb[u].x, wa[u].y, wb[u].y, xv[u][m].x, xv[u][m].y);
        mma_16816(c1[m], wa[u].z, wb[u].z, wa[u].w, wb[u].w, xv[u][m].z, xv[u][m].w);
      }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m) {
    red[warp][g][m * 8 + 2 * t] = c0[m][0] + c1[m][0];
    red[warp][g][m * 8 + 2 * t + 1] = c0[m][1] + c1[m][1];
    red[warp][g + 8][m * 8 + 2 * t] = c0[m][2] + c1[m][2];
    red[warp][g + 8][m * 8 + 2 * t + 1] = c0[m][3] + c1[m][3];
  }
  __syncthreads();
  const int rows = (kMvWarps / ks) * 16;
  for (int e = threadIdx.x; e < rows * 8 * MT; e += kMvWarps * 32) {
    const int r = e % rows, m = e / rows, n = blockIdx.x * rows + r;
    if (n >= a.N || m >= M) continue;
    float v = 0.f;
    for (int p = 0; p < ks; ++p) v += red[(r >> 4) * ks + p][r & 15][m];
    if (a.bias != nullptr) v += __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(a.bias)[n]);
    if (a.act_tanh) v = tanhf(v);
    const size_t o = blockIdx.z * a.ob + (size_t)(m0 + m) * a.ldo + n;
    if (a.accumulate) reinterpret_cast<float*>(a.out)[o] += v;
    else if (a.out_f32) reinterpret_cast<float*>(a.out)[o] = v;
    else reinterpret_cast<__nv_bfloat16*>(a.out)[o] = __float2bfloat16_rn(v);
  }
}

static int launch_matvec_mma(MatvecArgs a, int batch, cudaStream_t stream) {
  const int nkb = (a.K + 31) / 32, tiles = (a.N + 15) / 16;
  a.ks = kMvWarps;
  while (a.ks > 1 && (nkb < 4 * a.ks || (long long)tiles * batch * ((a.M + 15) / 16) * a.ks > 64LL * kNumSMs)) a.ks /= 2;
  const int per = kMvWarps / a.ks;
  dim3 grid((tiles + per - 1) / per, (a.M + 15) / 16, batch);
  if (grid.y > 65535) return -2;
  if (a.M <= 8) matvec_mma_kernel<1><<<grid, kMvWarps * 32, 0, stream>>>(a);
  else matvec_mma_kernel<2><<<grid, kMvWarps * 32, 0, stream>>>(a);
  return launch_status();
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
// One warp per token: the `top` largest router logits (ties: the lower index); scores sigmoid(z), or the softmax over the
// chosen logits.  bias [E] (or null) is added to the logits first.
__global__ void moe_route_kernel(const float* __restrict__ z, const float* __restrict__ bias, int* __restrict__ idx,
                                 float* __restrict__ w, int n, int E, int top, int ldz, int softmax) {
  const int t = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  if (t >= n) return;
  const float* row = z + (size_t)t * ldz;
  uint32_t taken = 0;                                  // bit i: expert 32 i + lane
  float largest = 0.f, sum = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int be = 0x7fffffff;
    for (int i = 0; 32 * i + lane < E; ++i)
      if (!(taken >> i & 1)) {
        const float v = row[32 * i + lane] + (bias != nullptr ? bias[32 * i + lane] : 0.f);
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
      if (k == 0) largest = best;
      const float e = softmax ? expf(best - largest) : sigmoid_f(best);
      sum += e;
      idx[t * top + k] = be;
      w[t * top + k] = e;
    }
  }
  if (softmax && lane == 0)
    for (int k = 0; k < top; ++k) w[t * top + k] /= sum;
}

// For slot = token * top + k, a warp multiplies two weight rows of expert e = idx[slot] with the token:
//   GLU false  hidden units f0, f0 + 1 of up [E, F, W]:  hid[slot][f] = (w_slot relu(up_e[f] . h))^2
//   GLU true   the gate and up rows of one hidden unit of [E, 2 F, W], which alternate in blocks of `block` rows:
//              hid[slot][f] = w_slot silu(gate_e[f] . h) (up_e[f] . h)
template <typename T, bool VEC, bool GLU>
__global__ void __launch_bounds__(256) moe_up_kernel(const T* __restrict__ h, const T* __restrict__ up,
                                                     const int* __restrict__ idx, const float* __restrict__ wgt,
                                                     T* __restrict__ hid, int top, int F, int W, int block) {
  const int slot = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int f0 = (blockIdx.x * 8 + warp) * (GLU ? 1 : 2);
  if (f0 >= F) return;
  const T* x = h + (size_t)(slot / top) * W;
  const T* u0 = GLU ? up + ((size_t)idx[slot] * 2 * F + (size_t)(f0 / block) * 2 * block + f0 % block) * W
                    : up + ((size_t)idx[slot] * F + f0) * W;
  const bool two = GLU || f0 + 1 < F;
  const size_t second = GLU ? (size_t)block * W : (two ? W : 0);
  float a0 = 0.f, a1 = 0.f;
#pragma unroll 2
  for (int k = lane * 8; k < W; k += 256) {
    float xf[8], w0[8], w1[8];
    if (VEC) {
      load_v<8>(x + k, xf);
      load_v<8>(u0 + k, w0);
      load_v<8>(u0 + second + k, w1);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const bool in = k + j < W;
        xf[j] = in ? to_f<T>(x[k + j]) : 0.f;
        w0[j] = in ? to_f<T>(u0[k + j]) : 0.f;
        w1[j] = in ? to_f<T>(u0[second + k + j]) : 0.f;
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
    if (GLU) {
      hid[(size_t)slot * F + f0] = from_f<T>(s * silu_f(a0) * a1);
      return;
    }
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
  if (is_bf16 && vec) return launch_matvec_mma(a, batch, stream);
  return is_bf16 ? dispatch_matvec<__nv_bfloat16>(a, batch, vec, stream) : dispatch_matvec<float>(a, batch, vec, stream);
}

ELL_API int ell_moe_route(const float* z, const float* bias, int* idx, float* w, int n, int E, int top, int ldz, int softmax,
                          cudaStream_t stream) {
  if (n <= 0) return 0;
  if (E > 1024 || top > E || top < 1) return -2;
  moe_route_kernel<<<(n + 7) / 8, 256, 0, stream>>>(z, bias, idx, w, n, E, top, ldz, softmax);
  return launch_status();
}

// acc [n, W] fp32 += experts; up [E, F, W], down [E, W, F]; hid: scratch [n * top, F] of the activation type.
// glu_block > 0: gated experts, up [E, 2 F, W] with gate and up rows in alternating blocks of glu_block (a divisor of F).
ELL_API int ell_moe_rows(const void* h, const void* up, const void* down, const int* idx, const float* w, void* hid,
                         float* acc, int n, int top, int F, int W, int glu_block, int is_bf16, cudaStream_t stream) {
  if (n <= 0) return 0;
  if ((long long)n * top > 65535) return -2;
  const bool v = F % 8 == 0 && W % 8 == 0 && aligned_to(h, 16) && aligned_to(up, 16) && aligned_to(down, 16) && aligned_to(hid, 16);
  if (glu_block < 0 || (glu_block > 0 && F % glu_block)) return -2;
  dim3 gu(glu_block ? (F + 7) / 8 : (F + 15) / 16, n * top), gd((W + 15) / 16, n);
#define ELL_MOE_ROWS(T, V)                                                                                          \
  if (glu_block) moe_up_kernel<T, V, true><<<gu, 256, 0, stream>>>((const T*)h, (const T*)up, idx, w, (T*)hid, top, F, W, glu_block); \
  else moe_up_kernel<T, V, false><<<gu, 256, 0, stream>>>((const T*)h, (const T*)up, idx, w, (T*)hid, top, F, W, 1); \
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
