// Elementwise and short-reduction kernels of the hybrid decoder layers (inference): scaled embedding (with a table of
// token pairs) into the fp32 stream, the dynamic-tanh norm, layer norms that share their statistics, gated activations,
// token shift, head norm with gate, key/value cache writes, the rotations and the norm of latent attention.
//
// Templated on the activation type (bf16 for serving, fp32 for exact runs); every value is computed in fp32.  Compiled
// without fast-math: tanh, exp and the divisions are the accurate ones, the fp32 runs depend on them.
#include "vec.cuh"

namespace ell {

template <typename T, int V>
__global__ void embed_scaled_kernel(const long long* __restrict__ ids, const T* __restrict__ table,
                                    float* __restrict__ out, int n, int W, long long rows, float scale,
                                    int* __restrict__ err) {
  const int wv = W / V;
  const long long total = (long long)n * wv;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / wv), c = (int)(i % wv) * V;
    const long long id = ids[t];
    float f[V];
    if (id < 0 || id >= rows) {
      atomicCAS(err, 0, 31);
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] = 0.f;
    } else {
      load_v<V>(table + id * W + c, f);
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] *= scale;
    }
    store_v<V>(out + (size_t)t * W + c, f);
  }
}

// y = tanh(alpha x) w + b; then x += add (the bias of the feed-forward that will accumulate into x), if given.
template <typename T, int V>
__global__ void dynamic_tanh_kernel(float* __restrict__ x, const float* __restrict__ alpha, const float* __restrict__ w,
                                    const float* __restrict__ b, const T* __restrict__ add, T* __restrict__ y, int n, int W) {
  const int wv = W / V;
  const long long total = (long long)n * wv;
  const float al = *alpha;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int c = (int)(i % wv) * V;
    float xv[V], wf[V], bf[V], o[V];
    load_v<V>(x + i * V, xv);
    load_v<V>(w + c, wf);
    load_v<V>(b + c, bf);
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] = tanhf(al * xv[j]) * wf[j] + bf[j];
    store_v<V>(y + i * V, o);
    if (add != nullptr) {
      load_v<V>(add + c, bf);
#pragma unroll
      for (int j = 0; j < V; ++j) xv[j] += bf[j];
      store_v<V>(x + i * V, xv);
    }
  }
}

enum Act { kActSilu = 0, kActGeluTanh = 1 };

template <typename T, int V>
__global__ void glu_kernel(const T* __restrict__ gu, T* __restrict__ out, int n, int F, int ld, int act) {
  const int fv = F / V;
  const long long total = (long long)n * fv;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / fv), c = (int)(i % fv) * V;
    float g[V], u[V];
    load_v<V>(gu + (size_t)t * ld + c, g);
    load_v<V>(gu + (size_t)t * ld + F + c, u);
#pragma unroll
    for (int j = 0; j < V; ++j) u[j] *= act == kActSilu ? silu_f(g[j]) : gelu_tanh_f(g[j]);
    store_v<V>(out + (size_t)t * F + c, u);
  }
}

// out = sigmoid(z[t]) relu(x)^2
template <typename T, int V>
__global__ void relu2_scaled_kernel(const T* __restrict__ x, const float* __restrict__ z, T* __restrict__ out, int n,
                                    int F, int ld, int ldz) {
  const int fv = F / V;
  const long long total = (long long)n * fv;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / fv), c = (int)(i % fv) * V;
    float f[V];
    load_v<V>(x + (size_t)t * ld + c, f);
    const float s = sigmoid_f(z[(size_t)t * ldz]);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float r = fmaxf(f[j], 0.f);
      f[j] = s * r * r;
    }
    store_v<V>(out + (size_t)t * F + c, f);
  }
}

template <typename T>
__global__ void tanh_cast_kernel(const float* __restrict__ x, T* __restrict__ y, int n, int N, int ldx) {
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < (long long)n * N;
       i += (long long)gridDim.x * blockDim.x)
    y[i] = from_f<T>(tanhf(x[(i / N) * ldx + i % N]));
}

// z = exp(-exp(z + w0[column]))
__global__ void wkv_decay_kernel(float* __restrict__ z, const float* __restrict__ w0, long long total, int C) {
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x)
    z[i] = expf(-expf(z[i] + w0[i % C]));
}

// out[c][t] = h[t] + (h[t-1] - h[t]) * mu[c].  Block (columns, chunk of tokens, sequence); a thread walks the tokens of
// its columns.  The row before a sequence's first one is zero, or its slot's `last` row when it goes on; chunk 0 is the
// only one to touch `last`, so it can replace it by the sequence's last row (h is complete) after reading it.
template <typename T, int V>
__global__ void token_mix_kernel(const T* __restrict__ h, const float* __restrict__ mu, T* __restrict__ out,
                                 const int* __restrict__ cu, const int* __restrict__ slots, const int* __restrict__ pos0,
                                 T* __restrict__ last, int W, int nmix, int n, int chunk) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= W) return;
  const int s = blockIdx.z, a = cu[s], b = cu[s + 1];
  int t0 = a + blockIdx.y * chunk;
  const int t1 = min(t0 + chunk, b);
  if (t0 >= t1) return;
  float prev[V];
  if (t0 > a) {
    load_v<V>(h + (size_t)(t0 - 1) * W + c, prev);
  } else {
#pragma unroll
    for (int j = 0; j < V; ++j) prev[j] = 0.f;
    if (last != nullptr) {
      T* l = last + (size_t)slots[s] * W + c;
      if (pos0[s] > 0) load_v<V>(l, prev);
      float nl[V];
      load_v<V>(h + (size_t)(b - 1) * W + c, nl);
      store_v<V>(l, nl);
    }
  }
  for (int t = t0; t < t1; ++t) {
    float x[V];
    load_v<V>(h + (size_t)t * W + c, x);
    for (int m = 0; m < nmix; ++m) {
      float mv[V], o[V];
      load_v<V>(mu + (size_t)m * W + c, mv);
#pragma unroll
      for (int j = 0; j < V; ++j) o[j] = x[j] + (prev[j] - x[j]) * mv[j];
      store_v<V>(out + ((size_t)m * n + t) * W + c, o);
    }
#pragma unroll
    for (int j = 0; j < V; ++j) prev[j] = x[j];
  }
}

// One warp per (token, head): y = o / rms(o) * w * act(gate).  IT pieces of V elements a lane are kept in registers, all
// loads ahead of the reduction (IT = 0: any head size, read twice).
template <typename T, int V, int IT>
__device__ __forceinline__ void head_norm_gate_row(const float* orow, const float* w, const T* gate, T* y, int dv,
                                                   int silu_gate, float eps, int lane) {
  if (IT > 0) {
    float f[IT > 0 ? IT : 1][V], g[IT > 0 ? IT : 1][V];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < IT; ++i) {
      const int c = (i * 32 + lane) * V;
      if (c < dv) {
        load_v<V>(orow + c, f[i]);
        load_v<V>(gate + c, g[i]);
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) f[i][j] = 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < IT; ++i)
#pragma unroll
      for (int j = 0; j < V; ++j) ss += f[i][j] * f[i][j];
    const float r = 1.f / sqrtf(warp_sum(ss) / dv + eps);
#pragma unroll
    for (int i = 0; i < IT; ++i) {
      const int c = (i * 32 + lane) * V;
      if (c < dv) {
        float wv[V];
        load_v<V>(w + c, wv);
#pragma unroll
        for (int j = 0; j < V; ++j) f[i][j] = f[i][j] * r * wv[j] * (silu_gate ? silu_f(g[i][j]) : sigmoid_f(g[i][j]));
        store_v<V>(y + c, f[i]);
      }
    }
  } else {
    float ss = 0.f;
    for (int c = lane * V; c < dv; c += 32 * V) {
      float f[V];
      load_v<V>(orow + c, f);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += f[j] * f[j];
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / dv + eps);
    for (int c = lane * V; c < dv; c += 32 * V) {
      float f[V], g[V], wv[V];
      load_v<V>(orow + c, f);
      load_v<V>(gate + c, g);
      load_v<V>(w + c, wv);
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] = f[j] * r * wv[j] * (silu_gate ? silu_f(g[j]) : sigmoid_f(g[j]));
      store_v<V>(y + c, f);
    }
  }
}

template <typename T, int V>
__global__ void head_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ w, const T* __restrict__ gate,
                                      T* __restrict__ y, int n, int H, int dv, int w_per_head, int ldg, int silu_gate,
                                      float eps) {
  const int warps = blockDim.x >> 5, lane = threadIdx.x & 31;
  for (long long i = blockIdx.x * (long long)warps + (threadIdx.x >> 5); i < (long long)n * H; i += (long long)gridDim.x * warps) {
    const int t = (int)(i / H), hd = (int)(i % H);
    const float* orow = o + (size_t)i * dv;
    const float* wrow = w + (w_per_head ? hd * dv : 0);
    const T* grow = gate + (size_t)t * ldg + (size_t)hd * dv;
    T* yrow = y + (size_t)i * dv;
    if (V == 4 && dv <= 128) head_norm_gate_row<T, V, 1>(orow, wrow, grow, yrow, dv, silu_gate, eps, lane);
    else if (V == 4 && dv <= 256) head_norm_gate_row<T, V, 2>(orow, wrow, grow, yrow, dv, silu_gate, eps, lane);
    else head_norm_gate_row<T, V, 0>(orow, wrow, grow, yrow, dv, silu_gate, eps, lane);
  }
}

// Token t's keys and values go to cache row kv_base[t] + kv_len[t] - 1.
template <typename T, int V>
__global__ void kv_append_kernel(const T* __restrict__ k, const T* __restrict__ v, T* __restrict__ kc, T* __restrict__ vc,
                                 const int* __restrict__ base, const int* __restrict__ len, int n, int dk, int dv, int ldk,
                                 int ldv) {
  const int per = (dk + dv) / V;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < (long long)n * per;
       i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / per), c = (int)(i % per) * V;
    const size_t row = (size_t)base[t] + len[t] - 1;
    float f[V];
    if (c < dk) {
      load_v<V>(k + (size_t)t * ldk + c, f);
      store_v<V>(kc + row * dk + c, f);
    } else {
      load_v<V>(v + (size_t)t * ldv + c - dk, f);
      store_v<V>(vc + row * dv + c - dk, f);
    }
  }
}

// out[t] = table[id] * scale + pairs[(previous id * mul_prev + id * mul_cur) mod buckets]; a sequence's first token takes
// row `buckets`.  One CTA per token.  The previous token is the row before, or, for the first row of a sequence that goes
// on, the entry before this one's in `hist` (token ids by position: row base[t] + len[t] - 1 is this token's, and is
// written).  hist null: every sequence starts in this batch.
template <typename T, int V>
__global__ void embed_pairs_kernel(const long long* __restrict__ ids, const T* __restrict__ table,
                                   const T* __restrict__ pairs, float* __restrict__ out, const int* __restrict__ row_start,
                                   const int* __restrict__ base, const int* __restrict__ len, int* __restrict__ hist, int W,
                                   long long rows, long long buckets, long long mul_prev, long long mul_cur, float scale,
                                   int* __restrict__ err) {
  const int t = blockIdx.x;
  const long long id = ids[t];
  const bool first_row = row_start[t] == t;
  const int place = hist != nullptr ? len[t] - 1 : 0;
  const size_t entry = hist != nullptr ? (size_t)base[t] + place : 0;
  long long prev = -1;
  if (!first_row) prev = ids[t - 1];
  else if (place > 0) prev = hist[entry - 1];
  const bool bad = id < 0 || id >= rows || prev >= rows;
  if (bad && threadIdx.x == 0) atomicCAS(err, 0, 31);
  const long long row = bad ? 0 : (prev < 0 ? buckets : (prev * mul_prev + id * mul_cur) % buckets);
  const T* a = table + (bad ? 0 : id) * W;
  const T* b = pairs + row * W;
  for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
    float f[V], g[V];
    load_v<V>(a + c, f);
    load_v<V>(b + c, g);
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] = bad ? 0.f : fmaf(f[j], scale, g[j]);
    store_v<V>(out + (size_t)t * W + c, f);
  }
  if (hist != nullptr && threadIdx.x == 0) hist[entry] = bad ? 0 : (int)id;
}

// Layer norms without a bias of one fp32 row, with one or two weights: y_i = (x - mean) / sqrt(variance + eps) * w_i.  One
// CTA per row; IT pieces of 4 columns a thread stay in registers (IT = 0: any width, re-read).
constexpr int kLnPairThreads = 256;

__device__ __forceinline__ float ln_block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < kLnPairThreads / 32; ++i) s += red[i];
  return s;
}

template <typename T, int IT>
__global__ void __launch_bounds__(kLnPairThreads)
layer_norms_kernel(const float* __restrict__ x, const float* __restrict__ w1, const float* __restrict__ w2,
                   T* __restrict__ y1, T* __restrict__ y2, int W, float eps) {
  __shared__ float red[2][kLnPairThreads / 32];
  const float* row = x + (size_t)blockIdx.x * W;
  T* o1 = y1 + (size_t)blockIdx.x * W;
  T* o2 = y2 + (size_t)blockIdx.x * W;
  if (IT > 0) {
    float f[IT > 0 ? IT : 1][4];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < IT; ++i) {
      const int c = (i * kLnPairThreads + threadIdx.x) * 4;
      if (c < W) load_v<4>(row + c, f[i]);
      else f[i][0] = f[i][1] = f[i][2] = f[i][3] = 0.f;
      s += (f[i][0] + f[i][1]) + (f[i][2] + f[i][3]);
    }
    const float mean = ln_block_sum(s, red[0]) / W;
    float q = 0.f;
#pragma unroll
    for (int i = 0; i < IT; ++i)
      if ((i * kLnPairThreads + threadIdx.x) * 4 < W)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          f[i][j] -= mean;
          q = fmaf(f[i][j], f[i][j], q);
        }
    const float r = 1.f / sqrtf(ln_block_sum(q, red[1]) / W + eps);
#pragma unroll
    for (int i = 0; i < IT; ++i) {
      const int c = (i * kLnPairThreads + threadIdx.x) * 4;
      if (c < W) {
        float w[4], o[4];
        load_v<4>(w1 + c, w);
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j] = f[i][j] * r * w[j];
        store_v<4>(o1 + c, o);
        if (w2 != nullptr) {
          load_v<4>(w2 + c, w);
#pragma unroll
          for (int j = 0; j < 4; ++j) o[j] = f[i][j] * r * w[j];
          store_v<4>(o2 + c, o);
        }
      }
    }
  } else {
    float s = 0.f;
    for (int c = threadIdx.x; c < W; c += kLnPairThreads) s += row[c];
    const float mean = ln_block_sum(s, red[0]) / W;
    float q = 0.f;
    for (int c = threadIdx.x; c < W; c += kLnPairThreads) q = fmaf(row[c] - mean, row[c] - mean, q);
    const float r = 1.f / sqrtf(ln_block_sum(q, red[1]) / W + eps);
    for (int c = threadIdx.x; c < W; c += kLnPairThreads) {
      const float v = (row[c] - mean) * r;
      o1[c] = from_f<T>(v * w1[c]);
      if (w2 != nullptr) o2[c] = from_f<T>(v * w2[c]);
    }
  }
}

// Latent attention between its input and its score products, in place on the projection rows z [n, ldz], whose columns
// are H queries of [dim unrotated, rot rotated], the latent of `rank`, one rotated key part:
//   rotated query parts -> z, or, with q_dst, to q_dst [n, H, q_stride]: neighbouring dimensions 2i, 2i+1 are a pair,
//     turned by the angle tables cos / sin [position, pairs]; dimensions past 2 * pairs pass unchanged
//   latent -> divided by its root mean square, times norm_w;  key part -> rotated
// Latent and key part also go to cache row base[t] + len[t] - 1 (rows of ldc), if there is a cache.
// One CTA per token; small enough that a dozen share an SM, since a token is a chain of dependent loads (its position,
// the angles there) around few bytes.
constexpr int kLatThreads = 128;
template <typename T, int V>
__global__ void __launch_bounds__(kLatThreads, 12)
latent_inputs_kernel(T* __restrict__ z, T* __restrict__ q_dst, T* __restrict__ cache, const float* __restrict__ norm_w,
                     const float* __restrict__ cosT, const float* __restrict__ sinT, const int* __restrict__ pos,
                     const int* __restrict__ base, const int* __restrict__ len, int H, int dim, int rot, int rank, int pairs,
                     int ldz, int q_stride, int ldc, float eps) {
  __shared__ float red[kLatThreads / 32];
  const int t = blockIdx.x;
  constexpr int VL = V == 8 ? 8 : 1;                    // pieces of the latent (any rank)
  T* row = z + (size_t)t * ldz;
  const int place = pos[t], qw = dim + rot;
  T* lat = row + (size_t)H * qw;
  T* kr = lat + rank;
  // the first piece of every thread stays in registers over the reduction
  float first[VL], ss = 0.f;
  const int c0 = threadIdx.x * VL;
  if (c0 < rank) load_v<VL>(lat + c0, first);
  else
#pragma unroll
    for (int j = 0; j < VL; ++j) first[j] = 0.f;
  T* crow = cache != nullptr ? cache + ((size_t)base[t] + len[t] - 1) * ldc : nullptr;
  // V consecutive dimensions from c on of the H query parts, then of the key part
  const int per = rot / V;
  for (int i = threadIdx.x; i < (H + 1) * per; i += kLatThreads) {
    const int h = i / per, c = (i - h * per) * V;
    const bool key = h == H;
    float f[V];
    load_v<V>((key ? kr : row + (size_t)h * qw + dim) + c, f);
    if (c / 2 < pairs) {
      const size_t at = (size_t)place * pairs + c / 2;
      if (V == 8) {                                     // pairs is a multiple of 4
        float cs[4], sn[4];
        load_v<4>(cosT + at, cs);
        load_v<4>(sinT + at, sn);
#pragma unroll
        for (int j = 0; j < V / 2; ++j) {
          const float a = f[2 * j], b = f[2 * j + 1];
          f[2 * j] = a * cs[j % 4] - b * sn[j % 4];
          f[2 * j + 1] = b * cs[j % 4] + a * sn[j % 4];
        }
      } else {
        const float a = f[0], b = f[1], cs = cosT[at], sn = sinT[at];
        f[0] = a * cs - b * sn;
        f[1] = b * cs + a * sn;
      }
    }
    store_v<V>((key ? kr : q_dst != nullptr ? q_dst + ((size_t)t * H + h) * q_stride : row + (size_t)h * qw + dim) + c, f);
    if (key && crow != nullptr) {
      if (V == 8) store_v<V>(crow + rank + c, f);
      else
#pragma unroll
        for (int j = 0; j < V; ++j) crow[rank + c + j] = from_f<T>(f[j]);
    }
  }
#pragma unroll
  for (int j = 0; j < VL; ++j) ss = fmaf(first[j], first[j], ss);
  for (int c = c0 + kLatThreads * VL; c < rank; c += kLatThreads * VL) {
    float f[VL];
    load_v<VL>(lat + c, f);
#pragma unroll
    for (int j = 0; j < VL; ++j) ss = fmaf(f[j], f[j], ss);
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < kLatThreads / 32; ++i) ss += red[i];
  const float r = 1.f / sqrtf(ss / rank + eps);
  for (int c = c0; c < rank; c += kLatThreads * VL) {
    float f[VL], w[VL];
    if (c == c0) {
#pragma unroll
      for (int j = 0; j < VL; ++j) f[j] = first[j];
    } else {
      load_v<VL>(lat + c, f);
    }
    load_v<VL>(norm_w + c, w);
#pragma unroll
    for (int j = 0; j < VL; ++j) f[j] = f[j] * r * w[j];
    store_v<VL>(lat + c, f);
    if (crow != nullptr) store_v<VL>(crow + c, f);
  }
}

}  // namespace ell

using namespace ell;

// `is_bf16` picks the activation type; `vec` is chosen so that every row start is aligned for it.
#define ELL_TV(cond_vec, KERNEL, GRID, BLOCK, ...)                                                     \
  do {                                                                                                 \
    if (is_bf16) {                                                                                     \
      using T = __nv_bfloat16;                                                                         \
      if (cond_vec) KERNEL<T, 4><<<GRID, BLOCK, 0, stream>>>(__VA_ARGS__);                             \
      else KERNEL<T, 1><<<GRID, BLOCK, 0, stream>>>(__VA_ARGS__);                                      \
    } else {                                                                                           \
      using T = float;                                                                                 \
      if (cond_vec) KERNEL<T, 4><<<GRID, BLOCK, 0, stream>>>(__VA_ARGS__);                             \
      else KERNEL<T, 1><<<GRID, BLOCK, 0, stream>>>(__VA_ARGS__);                                      \
    }                                                                                                  \
  } while (0)

ELL_API int ell_embed_scaled(const long long* ids, const void* table, float* out, int n, int W, long long rows,
                             float scale, int is_bf16, int* err, cudaStream_t stream) {
  if (n <= 0) return 0;
  const bool v = W % 4 == 0 && aligned_to(table, 16) && aligned_to(out, 16);
  const int g = grid_for((long long)n * (W / (v ? 4 : 1)), 256);
  ELL_TV(v, embed_scaled_kernel, g, 256, ids, (const T*)table, out, n, W, rows, scale, err);
  return launch_status();
}

ELL_API int ell_dynamic_tanh(float* x, const float* alpha, const float* w, const float* b, const void* add, void* y,
                             int n, int W, int is_bf16, cudaStream_t stream) {
  if (n <= 0) return 0;
  const bool v = W % 4 == 0 && aligned_to(x, 16) && aligned_to(y, 16) && aligned_to(w, 16) && aligned_to(b, 16) &&
                 aligned_to(add, 16);
  const int g = grid_for((long long)n * (W / (v ? 4 : 1)), 256);
  ELL_TV(v, dynamic_tanh_kernel, g, 256, x, alpha, w, b, (const T*)add, (T*)y, n, W);
  return launch_status();
}

// gu: rows of `ld` elements, gate columns [0, F), up columns [F, 2F); act 0 silu, 1 gelu (tanh form).
ELL_API int ell_glu(const void* gu, void* out, int n, int F, int ld, int act, int is_bf16, cudaStream_t stream) {
  if (n <= 0) return 0;
  const bool v = F % 4 == 0 && ld % 4 == 0 && aligned_to(gu, 16) && aligned_to(out, 16);
  const int g = grid_for((long long)n * (F / (v ? 4 : 1)), 256);
  ELL_TV(v, glu_kernel, g, 256, (const T*)gu, (T*)out, n, F, ld, act);
  return launch_status();
}

ELL_API int ell_relu2_scaled(const void* x, const float* z, void* out, int n, int F, int ld, int ldz, int is_bf16,
                             cudaStream_t stream) {
  if (n <= 0) return 0;
  const bool v = F % 4 == 0 && ld % 4 == 0 && aligned_to(x, 16) && aligned_to(out, 16);
  const int g = grid_for((long long)n * (F / (v ? 4 : 1)), 256);
  ELL_TV(v, relu2_scaled_kernel, g, 256, (const T*)x, z, (T*)out, n, F, ld, ldz);
  return launch_status();
}

ELL_API int ell_tanh_cast(const float* x, void* y, int n, int N, int ldx, int is_bf16, cudaStream_t stream) {
  if (n <= 0) return 0;
  const int g = grid_for((long long)n * N, 256);
  if (is_bf16) tanh_cast_kernel<__nv_bfloat16><<<g, 256, 0, stream>>>(x, (__nv_bfloat16*)y, n, N, ldx);
  else tanh_cast_kernel<float><<<g, 256, 0, stream>>>(x, (float*)y, n, N, ldx);
  return launch_status();
}

ELL_API int ell_wkv_decay(float* z, const float* w0, int n, int C, cudaStream_t stream) {
  if (n <= 0) return 0;
  wkv_decay_kernel<<<grid_for((long long)n * C, 256), 256, 0, stream>>>(z, w0, (long long)n * C, C);
  return launch_status();
}

// h [n, W] -> out [nmix, n, W].  last null: every sequence starts here and nothing is kept.
ELL_API int ell_token_mix(const void* h, const float* mu, void* out, const int* cu, const int* slots, const int* pos0,
                          void* last, int n, int n_seq, int max_len, int W, int nmix, int is_bf16, cudaStream_t stream) {
  if (n <= 0 || n_seq <= 0) return 0;
  if (n_seq > 65535) return -2;
  int chunk = 16;
  while ((max_len + chunk - 1) / chunk > 65535) chunk *= 2;
  const bool v = W % 4 == 0 && aligned_to(h, 16) && aligned_to(out, 16) && aligned_to(mu, 16) && aligned_to(last, 16);
  const int cols = W / (v ? 4 : 1), threads = cols >= 256 ? 256 : (cols + 31) / 32 * 32;
  dim3 g((cols + threads - 1) / threads, (max_len + chunk - 1) / chunk, n_seq);
  ELL_TV(v, token_mix_kernel, g, threads, (const T*)h, mu, (T*)out, cu, slots, pos0, (T*)last, W, nmix, n, chunk);
  return launch_status();
}

ELL_API int ell_head_norm_gate(const float* o, const float* w, const void* gate, void* y, int n, int H, int dv,
                               int w_per_head, int ldg, int silu_gate, float eps, int is_bf16, cudaStream_t stream) {
  if (n <= 0) return 0;
  const bool v = dv % 4 == 0 && ldg % 4 == 0 && aligned_to(o, 16) && aligned_to(w, 16) && aligned_to(gate, 16) &&
                 aligned_to(y, 16);
  const int g = grid_for((long long)n * H, 8, 64);
  ELL_TV(v, head_norm_gate_kernel, g, 256, o, w, (const T*)gate, (T*)y, n, H, dv, w_per_head, ldg, silu_gate, eps);
  return launch_status();
}

// k / v: rows of ldk / ldv elements holding dk = kv_heads * dim / dv = kv_heads * vdim values.
ELL_API int ell_kv_append(const void* k, const void* v_, void* kc, void* vc, const int* base, const int* len, int n,
                          int dk, int dv, int ldk, int ldv, int is_bf16, cudaStream_t stream) {
  if (n <= 0) return 0;
  const bool v = dk % 4 == 0 && dv % 4 == 0 && ldk % 4 == 0 && ldv % 4 == 0 && aligned_to(k, 16) && aligned_to(v_, 16) &&
                 aligned_to(kc, 16) && aligned_to(vc, 16);
  const int g = grid_for((long long)n * ((dk + dv) / (v ? 4 : 1)), 256);
  ELL_TV(v, kv_append_kernel, g, 256, (const T*)k, (const T*)v_, (T*)kc, (T*)vc, base, len, n, dk, dv, ldk, ldv);
  return launch_status();
}

// hist (and base / len): token ids by position, or null.
ELL_API int ell_embed_pairs(const long long* ids, const void* table, const void* pairs, float* out, const int* row_start,
                            const int* base, const int* len, int* hist, int n, int W, long long rows, long long buckets,
                            long long mul_prev, long long mul_cur, float scale, int is_bf16, int* err, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (buckets <= 0 || mul_prev < 0 || mul_cur < 0) return -2;
  const bool v = W % 4 == 0 && aligned_to(table, 16) && aligned_to(pairs, 16) && aligned_to(out, 16);
  ELL_TV(v, embed_pairs_kernel, n, 256, ids, (const T*)table, (const T*)pairs, out, row_start, base, len, hist, W, rows,
         buckets, mul_prev, mul_cur, scale, err);
  return launch_status();
}

// y1 = norm(x) w1, and with w2 also y2 = norm(x) w2.
ELL_API int ell_layer_norms(const float* x, const float* w1, const float* w2, void* y1, void* y2, int n, int W, float eps,
                            int is_bf16, cudaStream_t stream) {
  if (n <= 0) return 0;
  const bool v = W % 4 == 0 && W <= 8 * 4 * kLnPairThreads && aligned_to(x, 16) && aligned_to(w1, 16) &&
                 aligned_to(w2, 16) && aligned_to(y1, 16) && aligned_to(y2, 16);
  const int it = !v ? 0 : (W + 4 * kLnPairThreads - 1) / (4 * kLnPairThreads);
#define ELL_LN(IT)                                                                                                     \
  do {                                                                                                                 \
    if (is_bf16)                                                                                                       \
      layer_norms_kernel<__nv_bfloat16, IT><<<n, kLnPairThreads, 0, stream>>>(x, w1, w2, (__nv_bfloat16*)y1,           \
                                                                             (__nv_bfloat16*)y2, W, eps);             \
    else                                                                                                               \
      layer_norms_kernel<float, IT><<<n, kLnPairThreads, 0, stream>>>(x, w1, w2, (float*)y1, (float*)y2, W, eps);      \
  } while (0)
  if (it == 0) ELL_LN(0);
  else if (it == 1) ELL_LN(1);
  else if (it == 2) ELL_LN(2);
  else if (it <= 4) ELL_LN(4);
  else ELL_LN(8);
#undef ELL_LN
  return launch_status();
}

// q_dst null: queries are rotated in place.  cache null: nothing is kept.  rot is even.
ELL_API int ell_latent_inputs(void* z, void* q_dst, void* cache, const float* norm_w, const float* cosT, const float* sinT,
                              const int* pos, const int* base, const int* len, int n, int H, int dim, int rot, int rank,
                              int pairs, int ldz, int q_stride, int ldc, float eps, int is_bf16, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (rot % 2 || 2 * pairs > rot || rank < 1) return -2;
  const bool v = dim % 8 == 0 && rot % 8 == 0 && rank % 8 == 0 && pairs % 4 == 0 && aligned_to(cosT, 16) && aligned_to(sinT, 16) && ldz % 8 == 0 && q_stride % 8 == 0 && ldc % 8 == 0 &&
                 aligned_to(z, 16) && aligned_to(q_dst, 16) && aligned_to(cache, 16) && aligned_to(norm_w, 16);
#define ELL_LAT(T, V)                                                                                                   \
  latent_inputs_kernel<T, V><<<n, kLatThreads, 0, stream>>>((T*)z, (T*)q_dst, (T*)cache, norm_w, cosT, sinT, pos, base, \
                                                            len, H, dim, rot, rank, pairs, ldz, q_stride, ldc, eps)
  if (is_bf16) {
    if (v) ELL_LAT(__nv_bfloat16, 8);
    else ELL_LAT(__nv_bfloat16, 2);
  } else {
    if (v) ELL_LAT(float, 8);
    else ELL_LAT(float, 2);
  }
#undef ELL_LAT
  return launch_status();
}
