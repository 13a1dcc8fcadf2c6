// Elementwise and short-reduction kernels of the hybrid decoder layers (inference): scaled embedding into the fp32
// stream, the dynamic-tanh norm, gated activations, token shift, head norm with gate, key/value cache writes.
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
