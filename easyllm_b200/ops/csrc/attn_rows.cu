// Attention of single query rows over key/value rows: decoding from the cache, continued prompts, fp32 runs and head
// sizes the tcgen05 prefill kernel does not take.  GQA, value heads of their own size, ALiBi, a sink per head.
//
// Query row t sees the rows base[t] .. base[t] + len[t] - 1 of k [R, G, d] and v [R, G, dv] and sits at the last one.
// A CTA of 128 threads takes (row t, kv head, a range of keys) with all `rep` query heads of that kv head (in groups of
// at most 8), so every key and value is read once per group.  Tiles of KT keys and values come through two
// shared-memory stages (cp.async, the next tile in flight during the arithmetic).  Eight lanes share a key for the
// scores, the softmax runs on the KT scores of a head per warp, and for the weighted sum a thread owns eight value
// columns and a share of the tile's keys; the shares are added up once, at the end.  With more than one range per row a
// second kernel merges the partial (max, sum, accumulator) triples; the sink joins the denominator at the end, once.
#include "vec.cuh"

namespace ell {

constexpr int kArThreads = 128, kArRep = 8;   // kArRep: most query heads of a CTA (REP: 4 or 8)

struct AttnRowsArgs {
  const void *q, *k, *v;
  void* out;                      // [n, H, dv]
  float* part;                    // [n, H, splits, dv + 2] when splits > 1
  const int *base, *len;
  const float *sink, *slopes;
  int n, H, G, d, dv, ldq, ldk, ldv, splits, range;
  float scale;
};

// Shared memory: scaled queries [8][dp] | scores [8][KT] | statistics [8][4] | two stages of KT key rows, KT value rows.
struct ArLayout {
  int dp, krow, vrow, kgroups;    // padded key size; row strides in elements; key shares of the weighted sum
  int stage, bytes;               // elements of a stage; total bytes
};
__host__ __device__ inline ArLayout ar_layout(int d, int dv, int esz, int KT, int REP) {
  ArLayout l;
  l.dp = (d + 63) / 64 * 64;
  l.krow = l.dp + 16 / esz;
  const int oct = (dv + 7) / 8;
  l.vrow = oct * 8 + 16 / esz;
  l.kgroups = 1;
  while (2 * l.kgroups * oct <= kArThreads && 2 * l.kgroups <= KT / 4 && l.kgroups < 16) l.kgroups *= 2;
  l.stage = KT * (l.krow + l.vrow);
  const int head = (REP * l.dp + REP * KT + REP * 4) * 4;
  const int a = 2 * l.stage * esz, b = l.kgroups * REP * oct * 8 * 4;   // the sums reuse the stages
  l.bytes = head + (a > b ? a : b);
  return l;
}

template <typename T, int KT, int REP, bool VEC>
__global__ void __launch_bounds__(kArThreads) attn_rows_kernel(const AttnRowsArgs a) {
  extern __shared__ __align__(16) float sm[];
  const ArLayout L = ar_layout(a.d, a.dv, sizeof(T), KT, REP);
  const int t = blockIdx.x, rep = a.H / a.G, groups = (rep + REP - 1) / REP;
  const int g = blockIdx.y / groups, h0 = g * rep + (blockIdx.y % groups) * REP;
  const int nh = min(REP, g * rep + rep - h0);
  const int split = blockIdx.z, dp = L.dp, oct = (a.dv + 7) / 8;
  float* qs = sm;
  float* p = qs + REP * dp;
  float* stat = p + REP * KT;                    // max, sum, rescale
  T* stages = reinterpret_cast<T*>(stat + REP * 4);
  const int len = a.len[t];
  const size_t base = a.base[t];
  const int k0 = split * a.range, k1 = min(k0 + a.range, len);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // rows and columns the copies leave out must read as zero
  for (int i = threadIdx.x; i < 2 * L.stage * (int)sizeof(T) / 16; i += kArThreads)
    reinterpret_cast<uint4*>(stages)[i] = make_uint4(0, 0, 0, 0);
  for (int i = threadIdx.x; i < REP * dp; i += kArThreads) {
    const int h = i / dp, c = i % dp;
    qs[i] = h < nh && c < a.d
                ? to_f<T>(reinterpret_cast<const T*>(a.q)[(size_t)t * a.ldq + (size_t)(h0 + h) * a.d + c]) * a.scale : 0.f;
  }
  if (threadIdx.x < REP) {
    stat[threadIdx.x * 4] = -INFINITY;
    stat[threadIdx.x * 4 + 1] = 0.f;
  }
  __syncthreads();
  const T* kb = reinterpret_cast<const T*>(a.k) + base * a.ldk + (size_t)g * a.d;
  const T* vb = reinterpret_cast<const T*>(a.v) + base * a.ldv + (size_t)g * a.dv;
  auto load_tile = [&](int kt, int buf) {
    T* ks = stages + buf * L.stage;
    T* vs = ks + KT * L.krow;
    const int cnt = min(KT, k1 - kt);
    if (VEC) {
      constexpr int per = 16 / sizeof(T);
      const int kp = a.d / per, vp = a.dv / per;
      for (int i = threadIdx.x; i < cnt * kp; i += kArThreads) {
        const int r = i / kp, c = (i % kp) * per;
        cp_async16(ks + r * L.krow + c, kb + (size_t)(kt + r) * a.ldk + c);
      }
      for (int i = threadIdx.x; i < cnt * vp; i += kArThreads) {
        const int r = i / vp, c = (i % vp) * per;
        cp_async16(vs + r * L.vrow + c, vb + (size_t)(kt + r) * a.ldv + c);
      }
    } else {
      for (int i = threadIdx.x; i < cnt * a.d; i += kArThreads)
        ks[i / a.d * L.krow + i % a.d] = kb[(size_t)(kt + i / a.d) * a.ldk + i % a.d];
      for (int i = threadIdx.x; i < cnt * a.dv; i += kArThreads)
        vs[i / a.dv * L.vrow + i % a.dv] = vb[(size_t)(kt + i / a.dv) * a.ldv + i % a.dv];
    }
    cp_async_commit();
  };
  // weighted sum: this thread's eight columns and its share of a tile's keys
  const int my_oct = threadIdx.x % oct, my_share = threadIdx.x / oct, share = KT / L.kgroups;
  const bool adds = my_share < L.kgroups;
  float acc[REP][8];
#pragma unroll
  for (int h = 0; h < REP; ++h)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[h][j] = 0.f;
  const int l8 = lane & 7, grp = warp * 4 + (lane >> 3);          // 16 groups of 8 lanes
  constexpr int KJ = KT / 16;
  if (k0 < k1) load_tile(k0, 0);
  int buf = 0;
  for (int kt = k0; kt < k1; kt += KT, buf ^= 1) {
    if (kt + KT < k1) {
      load_tile(kt + KT, buf ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const T* ks = stages + buf * L.stage;
    const T* vs = ks + KT * L.krow;
    // scores: a group takes keys grp, grp + 16, ...
    float sc[REP][KJ];
#pragma unroll
    for (int h = 0; h < REP; ++h)
#pragma unroll
      for (int j = 0; j < KJ; ++j) sc[h][j] = 0.f;
    for (int c = l8 * 8; c < dp; c += 64) {
      float kv[KJ][8];
#pragma unroll
      for (int j = 0; j < KJ; ++j) load_v<8>(ks + (grp + 16 * j) * L.krow + c, kv[j]);
#pragma unroll
      for (int h = 0; h < REP; ++h) {
        if (h < nh) {
          const float4 q0 = *reinterpret_cast<const float4*>(qs + h * dp + c);
          const float4 q1 = *reinterpret_cast<const float4*>(qs + h * dp + c + 4);
#pragma unroll
          for (int j = 0; j < KJ; ++j) {
            float s = sc[h][j];
            s = fmaf(q0.x, kv[j][0], s); s = fmaf(q0.y, kv[j][1], s); s = fmaf(q0.z, kv[j][2], s); s = fmaf(q0.w, kv[j][3], s);
            s = fmaf(q1.x, kv[j][4], s); s = fmaf(q1.y, kv[j][5], s); s = fmaf(q1.z, kv[j][6], s); s = fmaf(q1.w, kv[j][7], s);
            sc[h][j] = s;
          }
        }
      }
    }
#pragma unroll
    for (int h = 0; h < REP; ++h) {
      if (h < nh) {
#pragma unroll
        for (int j = 0; j < KJ; ++j) {
          float s = sc[h][j];
          s += __shfl_xor_sync(0xffffffffu, s, 1);
          s += __shfl_xor_sync(0xffffffffu, s, 2);
          s += __shfl_xor_sync(0xffffffffu, s, 4);
          const int key = kt + grp + 16 * j;
          if (l8 == 0) {
            if (a.slopes != nullptr) s += a.slopes[h0 + h] * (float)(key - (len - 1));
            p[h * KT + grp + 16 * j] = key < k1 ? s : -INFINITY;
          }
        }
      }
    }
    __syncthreads();
    for (int h = warp; h < nh; h += 4) {
      float s[(KT + 31) / 32], mx = -INFINITY;
#pragma unroll
      for (int j = 0; j < (KT + 31) / 32; ++j) {
        s[j] = 32 * j + lane < KT ? p[h * KT + 32 * j + lane] : -INFINITY;
        mx = fmaxf(mx, s[j]);
      }
      const float m_old = stat[h * 4], m = fmaxf(m_old, warp_max(mx));   // finite: the tile has a key
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < (KT + 31) / 32; ++j) {
        const float e = expf(s[j] - m);
        sum += e;
        if (32 * j + lane < KT) p[h * KT + 32 * j + lane] = e;
      }
      sum = warp_sum(sum);
      if (lane == 0) {
        const float al = expf(m_old - m);
        stat[h * 4] = m;
        stat[h * 4 + 1] = stat[h * 4 + 1] * al + sum;
        stat[h * 4 + 2] = al;
      }
    }
    __syncthreads();
    if (adds) {
#pragma unroll
      for (int h = 0; h < REP; ++h) {
        if (h < nh) {
          const float al = stat[h * 4 + 2];
          if (al != 1.f) {
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[h][j] *= al;
          }
        }
      }
      const T* vp = vs + (size_t)(my_share * share) * L.vrow + my_oct * 8;
      for (int i = 0; i < share; i += 4) {
        float vv[4][8];
#pragma unroll
        for (int x = 0; x < 4; ++x) load_v<8>(vp + (i + x) * L.vrow, vv[x]);
#pragma unroll
        for (int h = 0; h < REP; ++h) {
          if (h < nh) {
            const float4 w = *reinterpret_cast<const float4*>(p + h * KT + my_share * share + i);
#pragma unroll
            for (int j = 0; j < 8; ++j)
              acc[h][j] = fmaf(w.w, vv[3][j], fmaf(w.z, vv[2][j], fmaf(w.y, vv[1][j], fmaf(w.x, vv[0][j], acc[h][j]))));
          }
        }
      }
    }
    __syncthreads();
  }
  // add the shares up: sums[share][head][column] over the stages' memory
  float* sums = reinterpret_cast<float*>(stages);
  if (adds) {
#pragma unroll
    for (int h = 0; h < REP; ++h)
      if (h < nh) store_v<8>(sums + ((my_share * REP + h) * oct + my_oct) * 8, acc[h]);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nh * a.dv; i += kArThreads) {
    const int h = i / a.dv, c = i % a.dv;
    float o = 0.f;
    for (int x = 0; x < L.kgroups; ++x) o += sums[(x * REP + h) * oct * 8 + c];
    const float m = stat[h * 4], l = stat[h * 4 + 1];
    if (a.splits == 1) {
      float den = l, f = 1.f;
      if (a.sink != nullptr) {
        const float sk = a.sink[h0 + h], mm = fmaxf(m, sk);
        f = expf(m - mm);
        den = l * f + expf(sk - mm);
      }
      reinterpret_cast<T*>(a.out)[((size_t)t * a.H + h0 + h) * a.dv + c] = from_f<T>(o * f / den);
    } else {
      float* pt = a.part + (((size_t)t * a.H + h0 + h) * a.splits + split) * (a.dv + 2);
      if (c == 0) {
        pt[0] = m;
        pt[1] = l;
      }
      pt[2 + c] = o;
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

// Query heads a CTA takes.
static int ar_rep(int rep) { return rep <= 4 ? 4 : kArRep; }

// Ranges per row: enough CTAs to fill the GPU a few times, about 256 keys each at least.
static int attn_rows_splits(int n, int H, int G, int max_len) {
  const int rep = H / G;
  const long long ctas = (long long)n * G * ((rep + ar_rep(rep) - 1) / ar_rep(rep));
  long long s = (4LL * kNumSMs + ctas - 1) / ctas;
  const long long most = (max_len + 255) / 256;
  if (s > most) s = most;
  if (s > 64) s = 64;
  return s < 1 ? 1 : (int)s;
}

template <typename T, int KT, int REP, bool VEC>
static int launch_attn_rows_kt(const AttnRowsArgs& a, dim3 grid, cudaStream_t stream) {
  const int bytes = ar_layout(a.d, a.dv, sizeof(T), KT, REP).bytes;
  auto kern = attn_rows_kernel<T, KT, REP, VEC>;
  static int configured = 0;
  if (bytes > configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return (int)e;
    configured = bytes;
  }
  kern<<<grid, kArThreads, bytes, stream>>>(a);
  if (a.splits > 1) attn_rows_merge_kernel<T><<<dim3(a.n, a.H), kArThreads, 0, stream>>>(a);
  return launch_status();
}

template <typename T, int REP>
static int launch_attn_rows(const AttnRowsArgs& a, dim3 grid, bool vec, cudaStream_t stream) {
  const bool small = ar_layout(a.d, a.dv, sizeof(T), 32, REP).bytes > 160 * 1024;      // very wide fp32 heads: short tiles
  if (small) return vec ? launch_attn_rows_kt<T, 16, REP, true>(a, grid, stream) : launch_attn_rows_kt<T, 16, REP, false>(a, grid, stream);
  return vec ? launch_attn_rows_kt<T, 32, REP, true>(a, grid, stream) : launch_attn_rows_kt<T, 32, REP, false>(a, grid, stream);
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
  if (H % G || dv > 512 || d > 512 || H > 65535) return -2;
  AttnRowsArgs a{q, k, v, out, part, base, len, sink, slopes, n, H, G, d, dv, ldq, ldk, ldv, 1, 0, scale};
  a.splits = attn_rows_splits(n, H, G, max_len);
  a.range = ((max_len + a.splits - 1) / a.splits + 63) / 64 * 64;
  if (a.splits > 1 && part == nullptr) return -2;
  const int rep = H / G, per = ar_rep(rep);
  dim3 grid(n, G * ((rep + per - 1) / per), a.splits);
  const int esz = is_bf16 ? 2 : 4;
  const bool vec = (d * esz) % 16 == 0 && (dv * esz) % 16 == 0 && (ldk * esz) % 16 == 0 && (ldv * esz) % 16 == 0 &&
                   aligned_to(k, 16) && aligned_to(v, 16);
  if (is_bf16)
    return per == 4 ? launch_attn_rows<__nv_bfloat16, 4>(a, grid, vec, stream) : launch_attn_rows<__nv_bfloat16, 8>(a, grid, vec, stream);
  return per == 4 ? launch_attn_rows<float, 4>(a, grid, vec, stream) : launch_attn_rows<float, 8>(a, grid, vec, stream);
}
