// Attention of single query rows over key/value rows: decoding from the cache, continued prompts, fp32 runs and head
// sizes the tcgen05 prefill kernel does not take.  GQA, value heads of their own size, ALiBi, a sink per head.
//
// Query row t sees the rows base[t] .. base[t] + len[t] - 1 of k [R, G, d] and v [R, G, dv] and sits at the last one.
// A CTA of 128 threads takes (row t, kv head, a range of keys) with all `rep` query heads of that kv head (in groups of
// at most 8), so every key and value is read once per group.  Tiles of 64 keys: eight lanes share a key for the scores
// (16-byte loads, queries from shared memory), the softmax runs on the 64 scores of a head per warp, and the threads
// own value columns for the weighted sum.  With more than one range per row a second kernel merges the partial
// (max, sum, accumulator) triples; the sink joins the denominator at the end, once.
#include "vec.cuh"

namespace ell {

constexpr int kArThreads = 128, kArKeys = 64, kArRep = 8;

struct AttnRowsArgs {
  const void *q, *k, *v;
  void* out;                      // [n, H, dv]
  float* part;                    // [n, H, splits, dv + 2] when splits > 1
  const int *base, *len;
  const float *sink, *slopes;
  int n, H, G, d, dv, ldq, ldk, ldv, splits, range;
  float scale;
};

template <typename T, bool VEC>
__global__ void __launch_bounds__(kArThreads) attn_rows_kernel(const AttnRowsArgs a) {
  extern __shared__ float sm[];
  const int t = blockIdx.x, rep = a.H / a.G, groups = (rep + kArRep - 1) / kArRep;
  const int g = blockIdx.y / groups, h0 = g * rep + (blockIdx.y % groups) * kArRep;
  const int nh = min(kArRep, g * rep + rep - h0);
  const int split = blockIdx.z;
  const int dp = (a.d + 63) / 64 * 64;
  float* qs = sm;                                   // [nh][dp]
  float* p = qs + kArRep * dp;                      // [nh][kArKeys]
  float* stat = p + kArRep * kArKeys;               // [nh][4]: max, sum, rescale
  const int len = a.len[t];
  const size_t base = a.base[t];
  const int k0 = split * a.range, k1 = min(k0 + a.range, len);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < nh * dp; i += kArThreads) {
    const int h = i / dp, c = i % dp;
    qs[i] = c < a.d ? to_f<T>(reinterpret_cast<const T*>(a.q)[(size_t)t * a.ldq + (size_t)(h0 + h) * a.d + c]) * a.scale : 0.f;
  }
  if (threadIdx.x < nh) {
    stat[threadIdx.x * 4] = -INFINITY;
    stat[threadIdx.x * 4 + 1] = 0.f;
  }
  // value columns of this thread: c = threadIdx.x + 128 j, up to 4 per pass (dv <= 512)
  float acc[kArRep][4];
#pragma unroll
  for (int h = 0; h < kArRep; ++h)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[h][j] = 0.f;
  __syncthreads();
  const T* kb = reinterpret_cast<const T*>(a.k) + base * a.ldk + (size_t)g * a.d;
  const T* vb = reinterpret_cast<const T*>(a.v) + base * a.ldv + (size_t)g * a.dv;
  const int l8 = lane & 7, grp = warp * 4 + (lane >> 3);          // 16 groups of 8 lanes
  for (int kt = k0; kt < k1; kt += kArKeys) {
    // scores: group takes keys grp, grp + 16, grp + 32, grp + 48 of the tile
    float sc[kArRep][4];
#pragma unroll
    for (int h = 0; h < kArRep; ++h)
#pragma unroll
      for (int j = 0; j < 4; ++j) sc[h][j] = 0.f;
    for (int c = l8 * 8; c < dp; c += 64) {
      float kv[4][8];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int key = kt + grp + 16 * j;
        const T* kp = kb + (size_t)key * a.ldk + c;
        if (key < k1 && VEC && c + 7 < a.d) {
          load_v<8>(kp, kv[j]);
        } else {
#pragma unroll
          for (int i = 0; i < 8; ++i) kv[j][i] = key < k1 && c + i < a.d ? to_f<T>(kp[i]) : 0.f;
        }
      }
#pragma unroll
      for (int h = 0; h < kArRep; ++h) {
        if (h < nh) {
          const float4 q0 = *reinterpret_cast<const float4*>(qs + h * dp + c);
          const float4 q1 = *reinterpret_cast<const float4*>(qs + h * dp + c + 4);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            float s = sc[h][j];
            s = fmaf(q0.x, kv[j][0], s); s = fmaf(q0.y, kv[j][1], s); s = fmaf(q0.z, kv[j][2], s); s = fmaf(q0.w, kv[j][3], s);
            s = fmaf(q1.x, kv[j][4], s); s = fmaf(q1.y, kv[j][5], s); s = fmaf(q1.z, kv[j][6], s); s = fmaf(q1.w, kv[j][7], s);
            sc[h][j] = s;
          }
        }
      }
    }
#pragma unroll
    for (int h = 0; h < kArRep; ++h) {
      if (h < nh) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          float s = sc[h][j];
          s += __shfl_xor_sync(0xffffffffu, s, 1);
          s += __shfl_xor_sync(0xffffffffu, s, 2);
          s += __shfl_xor_sync(0xffffffffu, s, 4);
          const int key = kt + grp + 16 * j;
          if (l8 == 0) {
            if (a.slopes != nullptr) s += a.slopes[h0 + h] * (float)(key - (len - 1));
            p[h * kArKeys + grp + 16 * j] = key < k1 ? s : -INFINITY;
          }
        }
      }
    }
    __syncthreads();
    for (int h = warp; h < nh; h += 4) {
      const float s0 = p[h * kArKeys + lane], s1 = p[h * kArKeys + 32 + lane];
      const float m_old = stat[h * 4], m = fmaxf(m_old, warp_max(fmaxf(s0, s1)));   // finite: the tile has a key
      const float e0 = expf(s0 - m), e1 = expf(s1 - m);
      p[h * kArKeys + lane] = e0;
      p[h * kArKeys + 32 + lane] = e1;
      const float sum = warp_sum(e0 + e1);
      if (lane == 0) {
        const float al = expf(m_old - m);
        stat[h * 4] = m;
        stat[h * 4 + 1] = stat[h * 4 + 1] * al + sum;
        stat[h * 4 + 2] = al;
      }
    }
    __syncthreads();
    const int cnt = min(kArKeys, k1 - kt);
#pragma unroll
    for (int h = 0; h < kArRep; ++h) {
      if (h < nh) {
        const float al = stat[h * 4 + 2];
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[h][j] *= al;
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = threadIdx.x + kArThreads * j;
      if (c < a.dv) {
        const T* vp = vb + (size_t)kt * a.ldv + c;
        int i = 0;
        for (; i + 4 <= cnt; i += 4) {
          float vv[4];
#pragma unroll
          for (int x = 0; x < 4; ++x) vv[x] = to_f<T>(vp[(size_t)(i + x) * a.ldv]);
#pragma unroll
          for (int h = 0; h < kArRep; ++h) {
            if (h < nh) {
              const float4 w = *reinterpret_cast<const float4*>(p + h * kArKeys + i);
              acc[h][j] = fmaf(w.x, vv[0], acc[h][j]); acc[h][j] = fmaf(w.y, vv[1], acc[h][j]);
              acc[h][j] = fmaf(w.z, vv[2], acc[h][j]); acc[h][j] = fmaf(w.w, vv[3], acc[h][j]);
            }
          }
        }
        for (; i < cnt; ++i) {
          const float vv = to_f<T>(vp[(size_t)i * a.ldv]);
#pragma unroll
          for (int h = 0; h < kArRep; ++h)
            if (h < nh) acc[h][j] = fmaf(p[h * kArKeys + i], vv, acc[h][j]);
        }
      }
    }
    __syncthreads();
  }
  // results
#pragma unroll
  for (int h = 0; h < kArRep; ++h) {
    if (h >= nh) continue;
    const float m = stat[h * 4], l = stat[h * 4 + 1];
    if (a.splits == 1) {
      float den = l, f = 1.f;
      if (a.sink != nullptr) {
        const float sk = a.sink[h0 + h], mm = fmaxf(m, sk);
        f = expf(m - mm);
        den = l * f + expf(sk - mm);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int c = threadIdx.x + kArThreads * j;
        if (c < a.dv) reinterpret_cast<T*>(a.out)[((size_t)t * a.H + h0 + h) * a.dv + c] = from_f<T>(acc[h][j] * f / den);
      }
    } else {
      float* pt = a.part + (((size_t)t * a.H + h0 + h) * a.splits + split) * (a.dv + 2);
      if (threadIdx.x == 0) {
        pt[0] = m;
        pt[1] = l;
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int c = threadIdx.x + kArThreads * j;
        if (c < a.dv) pt[2 + c] = acc[h][j];
      }
    }
  }
}

// One CTA per (row, head): merge the ranges' triples.  Empty ranges carry max = -inf, sum = 0.
template <typename T>
__global__ void __launch_bounds__(kArThreads) attn_rows_merge_kernel(const AttnRowsArgs a) {
  const int t = blockIdx.x, h = blockIdx.y;
  const float* pt = a.part + ((size_t)t * a.H + h) * a.splits * (a.dv + 2);
  const int used = min(a.splits, (a.len[t] + a.range - 1) / a.range);
  float m = a.sink != nullptr ? a.sink[h] : -INFINITY;
  for (int s = 0; s < used; ++s) m = fmaxf(m, pt[(size_t)s * (a.dv + 2)]);
  float den = a.sink != nullptr ? expf(a.sink[h] - m) : 0.f;
  for (int s = 0; s < used; ++s) den += pt[(size_t)s * (a.dv + 2) + 1] * expf(pt[(size_t)s * (a.dv + 2)] - m);
  for (int c = threadIdx.x; c < a.dv; c += kArThreads) {
    float o = 0.f;
    for (int s = 0; s < used; ++s) o = fmaf(pt[(size_t)s * (a.dv + 2) + 2 + c], expf(pt[(size_t)s * (a.dv + 2)] - m), o);
    reinterpret_cast<T*>(a.out)[((size_t)t * a.H + h) * a.dv + c] = from_f<T>(o / den);
  }
}

// Ranges per row: enough CTAs to fill the GPU a few times, at least 128 keys each.
static int attn_rows_splits(int n, int H, int G, int max_len) {
  const int rep = H / G;
  const long long ctas = (long long)n * G * ((rep + kArRep - 1) / kArRep);
  long long s = (4LL * kNumSMs + ctas - 1) / ctas;
  const long long most = (max_len + 127) / 128;
  if (s > most) s = most;
  if (s > 64) s = 64;
  return s < 1 ? 1 : (int)s;
}

}  // namespace ell

using namespace ell;

// Scratch floats a call needs (0: none).
ELL_API long long ell_attn_rows_scratch(int n, int H, int G, int dv, int max_len) {
  const int s = attn_rows_splits(n, H, G, max_len);
  return s == 1 ? 0 : (long long)n * H * s * (dv + 2);
}

// Rows of ldq / ldk / ldv elements; max_len bounds len[] (it sets the number of ranges, longer rows would be cut).
ELL_API int ell_attn_rows(const void* q, const void* k, const void* v, void* out, float* part, const int* base,
                          const int* len, const float* sink, const float* slopes, int n, int H, int G, int d, int dv,
                          int ldq, int ldk, int ldv, int max_len, float scale, int is_bf16, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (H % G || dv > 4 * kArThreads || d > 512 || H > 65535) return -2;
  AttnRowsArgs a{q, k, v, out, part, base, len, sink, slopes, n, H, G, d, dv, ldq, ldk, ldv, 1, 0, scale};
  a.splits = attn_rows_splits(n, H, G, max_len);
  a.range = ((max_len + a.splits - 1) / a.splits + kArKeys - 1) / kArKeys * kArKeys;
  if (a.splits > 1 && part == nullptr) return -2;
  const int rep = H / G, dp = (d + 63) / 64 * 64;
  const size_t smem = (size_t)(kArRep * dp + kArRep * kArKeys + kArRep * 4) * 4;
  dim3 grid(n, G * ((rep + kArRep - 1) / kArRep), a.splits);
  const int esz = is_bf16 ? 2 : 4;
  const bool vec = d % 8 == 0 && (ldk * esz) % 16 == 0 && aligned_to(k, 16);
  if (is_bf16) {
    if (vec) attn_rows_kernel<__nv_bfloat16, true><<<grid, kArThreads, smem, stream>>>(a);
    else attn_rows_kernel<__nv_bfloat16, false><<<grid, kArThreads, smem, stream>>>(a);
    if (a.splits > 1) attn_rows_merge_kernel<__nv_bfloat16><<<dim3(n, H), kArThreads, 0, stream>>>(a);
  } else {
    if (vec) attn_rows_kernel<float, true><<<grid, kArThreads, smem, stream>>>(a);
    else attn_rows_kernel<float, false><<<grid, kArThreads, smem, stream>>>(a);
    if (a.splits > 1) attn_rows_merge_kernel<float><<<dim3(n, H), kArThreads, 0, stream>>>(a);
  }
  return launch_status();
}
