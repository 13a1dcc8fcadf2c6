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
// A window keeps the last `window` of a row's keys.  A gate multiplies head h's output of row t by sigmoid(gate[t][h]).
//
// Latent attention (one key row shared by all query heads, whose first dv columns are also the value, bf16) has a
// kernel of its own, attn_latent_kernel: the products run on mma.sync m16n8k16 over a key tile that is read once.
#include "sm100.cuh"
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
  int window;                     // keys a row sees at most (INT_MAX: all)
  const void* gate;               // [n, ldg] of the activation type, or null
  int ldg;
  int* err;                       // error word (latent kernel)
};

// Keys row t sees: the last min(len, window) of its rows.
struct RowKeys {
  size_t base;
  int len;
};
__device__ __forceinline__ RowKeys row_keys(const AttnRowsArgs& a, int t) {
  const int all = a.len[t], len = min(all, a.window);
  return {(size_t)a.base[t] + (all - len), len};
}
template <typename T>
__device__ __forceinline__ float row_gate(const AttnRowsArgs& a, int t, int h) {
  return a.gate == nullptr ? 1.f : sigmoid_f(to_f<T>(reinterpret_cast<const T*>(a.gate)[(size_t)t * a.ldg + h]));
}

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
  const RowKeys rk = row_keys(a, t);
  const int len = rk.len;
  const size_t base = rk.base;
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
      reinterpret_cast<T*>(a.out)[((size_t)t * a.H + h0 + h) * a.dv + c] = from_f<T>(o * f / den * row_gate<T>(a, t, h0 + h));
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

// One CTA per (row, head): merge the ranges' triples.  Empty ranges carry max = -inf, sum = 0.  The ranges' weights are
// formed once (a range a thread), then every thread sums its columns over the ranges with independent loads.
constexpr int kArMaxSplits = 64;
template <typename T>
__global__ void __launch_bounds__(kArThreads) attn_rows_merge_kernel(const AttnRowsArgs a) {
  __shared__ float weight[kArMaxSplits];
  const int t = blockIdx.x, h = blockIdx.y, step = a.dv + 2;
  const float* pt = a.part + ((size_t)t * a.H + h) * a.splits * step;
  const int used = min(a.splits, (row_keys(a, t).len + a.range - 1) / a.range);
  if (threadIdx.x < 32) {
    const int s0 = threadIdx.x, s1 = threadIdx.x + 32;
    const float m0 = s0 < used ? pt[(size_t)s0 * step] : -INFINITY, m1 = s1 < used ? pt[(size_t)s1 * step] : -INFINITY;
    const float l0 = s0 < used ? pt[(size_t)s0 * step + 1] : 0.f, l1 = s1 < used ? pt[(size_t)s1 * step + 1] : 0.f;
    const float sk = a.sink != nullptr ? a.sink[h] : -INFINITY;
    const float m = fmaxf(warp_max(fmaxf(m0, m1)), sk);            // finite: the first range has a key
    const float e0 = expf(m0 - m), e1 = expf(m1 - m);
    const float den = warp_sum(l0 * e0 + l1 * e1) + (a.sink != nullptr ? expf(sk - m) : 0.f);
    const float f = row_gate<T>(a, t, h) / den;
    weight[s0] = e0 * f;
    weight[s1] = e1 * f;
  }
  __syncthreads();
  T* out = reinterpret_cast<T*>(a.out) + ((size_t)t * a.H + h) * a.dv;
  if (a.dv % 2 == 0) {                                             // triples start at even places
    for (int c = threadIdx.x * 2; c < a.dv; c += 2 * kArThreads) {
      float2 o = make_float2(0.f, 0.f);
#pragma unroll 8
      for (int s = 0; s < used; ++s) {
        const float2 v = *reinterpret_cast<const float2*>(pt + (size_t)s * step + 2 + c);
        o.x = fmaf(v.x, weight[s], o.x);
        o.y = fmaf(v.y, weight[s], o.y);
      }
      out[c] = from_f<T>(o.x);
      out[c + 1] = from_f<T>(o.y);
    }
  } else {
    for (int c = threadIdx.x; c < a.dv; c += kArThreads) {
      float o = 0.f;
#pragma unroll 8
      for (int s = 0; s < used; ++s) o = fmaf(pt[(size_t)s * step + 2 + c], weight[s], o);
      out[c] = from_f<T>(o);
    }
  }
}

// ---- latent attention: all heads share one key row, its first dv columns are the value ---------------
// A CTA of 16 warps takes (row t, 16 * MT query heads, a range of keys).  Tiles of 64 key rows come through two
// shared-memory stages as TMA boxes of 64 columns (128-byte swizzle: ldmatrix meets no bank conflicts).
//   scores   a warp multiplies 16 heads with 32 keys over one of 8 / MT slices of the columns (k-steps of 16); the
//            slices' sums go to shared memory in fp32
//   softmax  a warp owns MT heads, 32 / MT lanes each; fp32 weights, their sum unrounded, the operand of P·V in bf16
//   values   warp w owns columns [w, w + 1) * dv / 16 of all heads; the value operand is the key tile itself (ldmatrix
//            with transposition); its rescaled accumulators stay in registers
constexpr int kAlWarps = 16, kAlKeys = 64, kAlPStride = kAlKeys + 8, kAlSStride = kAlKeys + 4, kAlMaxNt = 4;
constexpr int kAlSRows = 8 * 16;                 // slices of the score product x heads
constexpr int kAlErr = 14;

constexpr int kAlBoxBytes = kAlKeys * 128;             // [64 keys x 64 columns]
__host__ __device__ inline int al_krow(int d) { return (d + 15) / 16 * 16 + 8; }       // stride of a query row
static int al_bytes(int d, int MT) {
  return 1024 + 2 * ((d + 63) / 64) * kAlBoxBytes + 16 * MT * (al_krow(d) * 2 + kAlPStride * 2 + 16) +
         kAlSRows * kAlSStride * 4 + 32;
}
// Place of a 16-byte piece (8 columns) of a key row in a stage.
__device__ __forceinline__ uint32_t al_place(int row, int piece) {
  return (uint32_t)((piece >> 3) * kAlBoxBytes + row * 128 + (((piece & 7) ^ (row & 7)) << 4));
}

__device__ __forceinline__ void ldsm4(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void ldsm4_t(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int MT>
__global__ void __launch_bounds__(kAlWarps * 32)
attn_latent_kernel(const __grid_constant__ CUtensorMap tmK, const AttnRowsArgs a) {
  extern __shared__ uint8_t alsm_raw[];
  uint8_t* kv = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(alsm_raw) + 1023) & ~(uintptr_t)1023);
  constexpr int HM = 16 * MT;
  const int krow = al_krow(a.d), dp = krow - 8, boxes = (a.d + 63) / 64, stage_bytes = boxes * kAlBoxBytes;
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(kv + 2 * stage_bytes);
  __nv_bfloat16* ps = qs + HM * krow;
  float* ss = reinterpret_cast<float*>(ps + HM * kAlPStride);
  float* stat = ss + kAlSRows * kAlSStride;                  // max | sum | rescale, HM each
  uint64_t* full = reinterpret_cast<uint64_t*>(stat + 4 * HM);      // one barrier a stage
  int* gave_up = reinterpret_cast<int*>(full + 2);
  const int t = blockIdx.x, h0 = blockIdx.y * HM, nh = min(HM, a.H - h0), split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const RowKeys rk = row_keys(a, t);
  const int k0 = split * a.range, k1 = min(k0 + a.range, rk.len);
  const __nv_bfloat16* qb = reinterpret_cast<const __nv_bfloat16*>(a.q) + (size_t)t * a.ldq + (size_t)h0 * a.d;
  const int pieces = a.d / 8, padded = dp / 8;         // 16-byte pieces of a row
  const int tail = k1 > k0 ? (k1 - k0 - 1) % kAlKeys + 1 : kAlKeys, tiles = k1 > k0 ? (k1 - k0 + kAlKeys - 1) / kAlKeys : 0;
  // one thread: columns past d and rows past the tensor are zero-filled
  auto load_tile = [&](int kt, int buf) {
    sm100::mbar_expect_tx(&full[buf], (uint32_t)stage_bytes);
    for (int c = 0; c < boxes; ++c)
      sm100::tma_load_2d(kv + buf * stage_bytes + c * kAlBoxBytes, &tmK, &full[buf], c * 64, (int)rk.base + kt);
  };
  if (threadIdx.x == 0) {
    sm100::mbar_init(&full[0], 1);
    sm100::mbar_init(&full[1], 1);
    *gave_up = *(volatile int*)a.err;                  // an earlier kernel already failed: do not wait on anything
    sm100::fence_barrier_init();
    if (tiles > 0 && *gave_up == 0) load_tile(k0, 0);  // on its way while the queries come
  }
  // query rows and columns past the end read as zero
  for (int i = threadIdx.x; i < HM * padded; i += kAlWarps * 32) {
    const int h = i / padded, c = i % padded;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (h < nh && c < pieces) v = *reinterpret_cast<const uint4*>(qb + (size_t)h * a.d + c * 8);
    *reinterpret_cast<uint4*>(qs + h * krow + c * 8) = v;
  }
  if (threadIdx.x < HM) {
    stat[threadIdx.x] = -INFINITY;
    stat[HM + threadIdx.x] = 0.f;
    stat[2 * HM + threadIdx.x] = 1.f;
  }
  const int nt = (a.dv / 8 + kAlWarps - 1) / kAlWarps;         // 8-column pieces of a warp
  const int col0 = warp * nt * 8, mine = max(0, min(nt, (a.dv - col0) / 8));
  float acc[MT][kAlMaxNt][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < kAlMaxNt; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[m][n][i] = 0.f;
  const int g = lane >> 2, tq = lane & 3;
  const int l8 = lane & 7, quad = lane >> 3;
  __syncthreads();
  const bool dead = *gave_up != 0;
  constexpr int KS = 8 / MT;                             // column slices of the score product
  const int mt = MT == 1 ? 0 : warp >> 3, key0 = (warp & 1) * 32, slice = (warp >> 1) % KS;
  for (int it = 0; it < tiles && !dead; ++it) {
    const int buf = it & 1, kt = k0 + it * kAlKeys;
    uint8_t* ks = kv + buf * stage_bytes;
    if (threadIdx.x == 0 && it + 1 < tiles) load_tile(kt + kAlKeys, buf ^ 1);   // the end of the last step freed that stage
    if (!sm100::mbar_wait(&full[buf], (it >> 1) & 1, gave_up)) *(volatile int*)gave_up = 1;
    else if (it == tiles - 1)                            // rows past the range are other keys: their weight is 0, not their value
      for (int i = threadIdx.x; i < (kAlKeys - tail) * padded; i += kAlWarps * 32)
        *reinterpret_cast<uint4*>(ks + al_place(tail + i / padded, i % padded)) = make_uint4(0, 0, 0, 0);
    __syncthreads();
    if (*(volatile int*)gave_up) {
      if (threadIdx.x == 0) {
        atomicCAS(a.err, 0, kAlErr);
        const unsigned long long t0 = sm100::globaltimer_ns();          // copies still in flight land before the CTA ends
        while (sm100::globaltimer_ns() - t0 < 200000ull) {
        }
      }
      __syncthreads();
      break;                                             // uniform: every thread reads the flag after the barrier
    }
    // scores of 16 heads and 32 keys over this warp's slice of the columns
    {
      float sc[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) sc[n][i] = 0.f;
      const __nv_bfloat16* qrow = qs + (mt * 16 + (quad & 1) * 8 + l8) * krow + (quad >> 1) * 8;
      const int krow_i = key0 + (quad >> 1) * 8 + l8;
#pragma unroll 3
      for (int c = slice * 16; c < dp; c += KS * 16) {
        uint32_t a0[4], b0[4], b1[4];
        ldsm4(a0, qrow + c);
        const uint32_t at = al_place(krow_i, (c >> 3) + (quad & 1));       // 16 rows on: the same swizzle
        ldsm4(b0, ks + at);
        ldsm4(b1, ks + at + 16 * 128);
        mma_bf16(sc[0], a0, b0[0], b0[1]);
        mma_bf16(sc[1], a0, b0[2], b0[3]);
        mma_bf16(sc[2], a0, b1[0], b1[1]);
        mma_bf16(sc[3], a0, b1[2], b1[3]);
      }
      float* dst = ss + (slice * HM + mt * 16 + g) * kAlSStride + key0 + tq * 2;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        *reinterpret_cast<float2*>(dst + n * 8) = make_float2(sc[n][0], sc[n][1]);
        *reinterpret_cast<float2*>(dst + 8 * kAlSStride + n * 8) = make_float2(sc[n][2], sc[n][3]);
      }
    }
    __syncthreads();
    {
      constexpr int LH = 32 / MT, KL = kAlKeys / LH;       // lanes a head, keys a lane
      const int hh = warp * MT + lane / LH, key = (lane % LH) * KL;
      float sv[KL], mx = -INFINITY, sum = 0.f;
#pragma unroll
      for (int j = 0; j < KL; ++j) sv[j] = 0.f;
#pragma unroll
      for (int y = 0; y < KS; ++y) {
        const float* row = ss + (y * HM + hh) * kAlSStride + key;
#pragma unroll
        for (int j = 0; j < KL; j += 2) {
          const float2 v = *reinterpret_cast<const float2*>(row + j);
          sv[j] += v.x;
          sv[j + 1] += v.y;
        }
      }
#pragma unroll
      for (int j = 0; j < KL; ++j) {
        sv[j] = kt + key + j < k1 ? sv[j] * a.scale : -INFINITY;
        mx = fmaxf(mx, sv[j]);
      }
#pragma unroll
      for (int o = LH / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_old = stat[hh], m = fmaxf(m_old, mx);  // finite: the tile has a key
#pragma unroll
      for (int j = 0; j < KL; ++j) {
        sv[j] = expf(sv[j] - m);
        sum += sv[j];
      }
#pragma unroll
      for (int j = 0; j < KL; j += 2)
        *reinterpret_cast<__nv_bfloat162*>(ps + hh * kAlPStride + key + j) = __floats2bfloat162_rn(sv[j], sv[j + 1]);
#pragma unroll
      for (int o = LH / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      if (lane % LH == 0) {                                // its lanes have read the old maximum: the shuffles above
        const float al = expf(m_old - m);
        stat[hh] = m;
        stat[HM + hh] = stat[HM + hh] * al + sum;
        stat[2 * HM + hh] = al;
      }
    }
    __syncthreads();
    uint32_t pa[MT][kAlKeys / 16][4];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float r0 = stat[2 * HM + m * 16 + g], r1 = stat[2 * HM + m * 16 + g + 8];
#pragma unroll
      for (int n = 0; n < kAlMaxNt; ++n) {
        acc[m][n][0] *= r0;
        acc[m][n][1] *= r0;
        acc[m][n][2] *= r1;
        acc[m][n][3] *= r1;
      }
#pragma unroll
      for (int k = 0; k < kAlKeys / 16; ++k)
        ldsm4(pa[m][k], ps + (m * 16 + (quad & 1) * 8 + l8) * kAlPStride + k * 16 + (quad >> 1) * 8);
    }
#pragma unroll
    for (int n = 0; n < kAlMaxNt; ++n) {
      if (n < mine) {
#pragma unroll
        for (int k = 0; k < kAlKeys / 32; ++k) {         // 32 keys x 8 columns per ldmatrix
          uint32_t b[4];
          ldsm4_t(b, ks + al_place(k * 32 + quad * 8 + l8, col0 / 8 + n));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16(acc[m][n], pa[m][2 * k], b[0], b[1]);
            mma_bf16(acc[m][n], pa[m][2 * k + 1], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int hh = m * 16 + g + r * 8;
      if (hh >= nh) continue;
      const size_t th = (size_t)t * a.H + h0 + hh;
      const float l = stat[HM + hh];
      if (a.splits == 1) {
        const float f = row_gate<__nv_bfloat16>(a, t, h0 + hh) / l;
        __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(a.out) + th * a.dv + col0 + tq * 2;
#pragma unroll
        for (int n = 0; n < kAlMaxNt; ++n)
          if (n < mine)
            *reinterpret_cast<__nv_bfloat162*>(o + n * 8) = __floats2bfloat162_rn(acc[m][n][2 * r] * f, acc[m][n][2 * r + 1] * f);
      } else {
        float* pt = a.part + (th * a.splits + split) * (a.dv + 2);
        if (warp == 0 && tq == 0) {
          pt[0] = stat[hh];
          pt[1] = l;
        }
#pragma unroll
        for (int n = 0; n < kAlMaxNt; ++n)
          if (n < mine) *reinterpret_cast<float2*>(pt + 2 + col0 + n * 8 + tq * 2) = make_float2(acc[m][n][2 * r], acc[m][n][2 * r + 1]);
      }
    }
}

static int al_mt(int H) { return H > 16 ? 2 : 1; }

// Ranges per row of the latent kernel: one CTA an SM, at least one tile each.
static int attn_latent_splits(int n, int H, int max_len) {
  const long long ctas = (long long)n * ((H + 16 * al_mt(H) - 1) / (16 * al_mt(H)));
  long long s = kNumSMs / ctas;
  const long long most = (max_len + kAlKeys - 1) / kAlKeys;
  if (s > most) s = most;
  if (s > kArMaxSplits) s = kArMaxSplits;
  return s < 1 ? 1 : (int)s;
}

int make_tmap_bf16_2d(CUtensorMap* map, const void* ptr, uint64_t inner, uint64_t outer, uint64_t row_stride_bytes,
                      uint32_t box_inner, uint32_t box_outer);

template <int MT>
static int launch_attn_latent(const AttnRowsArgs& a, long long rows, cudaStream_t stream) {
  CUtensorMap tk;
  const int rc = make_tmap_bf16_2d(&tk, a.k, (uint64_t)a.d, (uint64_t)rows, (uint64_t)a.ldk * 2, 64, kAlKeys);
  if (rc) return rc;
  const int bytes = al_bytes(a.d, MT);
  static int configured = 0;
  if (bytes > configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_latent_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return (int)e;
    configured = bytes;
  }
  attn_latent_kernel<MT><<<dim3(a.n, (a.H + 16 * MT - 1) / (16 * MT), a.splits), kAlWarps * 32, bytes, stream>>>(tk, a);
  if (a.splits > 1) attn_rows_merge_kernel<__nv_bfloat16><<<dim3(a.n, a.H), kArThreads, 0, stream>>>(a);
  return launch_status();
}

// Shapes of the mma kernel; everything else runs on attn_rows_kernel.
static bool attn_latent_fits(const void* k, int d, int dv, int ldq, int ldk, int H) {
  return aligned_to(k, 16) && d % 8 == 0 && dv % 8 == 0 && dv <= d && dv <= 8 * kAlWarps * kAlMaxNt && ldq % 8 == 0 && ldk % 8 == 0 &&
         H <= 65535 && al_bytes(d, al_mt(H)) <= 227 * 1024;
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
  if (s > kArMaxSplits) s = kArMaxSplits;
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
// window: keys a row sees (<= 0: all).  gate: rows of ldg elements of the activation type, or null.
ELL_API int ell_attn_rows(const void* q, const void* k, const void* v, void* out, float* part, const int* base,
                          const int* len, const float* sink, const float* slopes, const void* gate, int n, int H, int G,
                          int d, int dv, int ldq, int ldk, int ldv, int ldg, int max_len, int window, float scale,
                          int is_bf16, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (H % G || dv > 8 * kArThreads || H > 65535) return -2;
  if (window <= 0) window = 0x7fffffff;
  if (max_len > window) max_len = window;
  AttnRowsArgs a{q, k, v, out, part, base, len, sink, slopes, n, H, G, d, dv, ldq, ldk, ldv, 1, 0, scale, window, gate, ldg, nullptr};
  a.splits = attn_rows_splits(n, H, G, max_len);
  a.range = ((max_len + a.splits - 1) / a.splits + 63) / 64 * 64;
  if (a.splits > 1 && part == nullptr) return -2;
  const int rep = H / G, per = ar_rep(rep);
  dim3 grid(n, G * ((rep + per - 1) / per), a.splits);
  const int esz = is_bf16 ? 2 : 4;
  if (ar_layout(d, dv, esz, 16, per).bytes > 227 * 1024) return -2;
  const bool vec = (d * esz) % 16 == 0 && (dv * esz) % 16 == 0 && (ldk * esz) % 16 == 0 && (ldv * esz) % 16 == 0 &&
                   aligned_to(k, 16) && aligned_to(v, 16);
  if (is_bf16)
    return per == 4 ? launch_attn_rows<__nv_bfloat16, 4>(a, grid, vec, stream) : launch_attn_rows<__nv_bfloat16, 8>(a, grid, vec, stream);
  return per == 4 ? launch_attn_rows<float, 4>(a, grid, vec, stream) : launch_attn_rows<float, 8>(a, grid, vec, stream);
}

// Latent attention: q [n, H, d] (rows of ldq), one key row [d] per position (`rows` rows of ldk) whose first dv columns are
// the value -> out [n, H, dv].  bf16 shapes the mma kernel takes run there, others on attn_rows.
ELL_API long long ell_attn_latent_scratch(const void* k, int n, int H, int d, int dv, int ldq, int ldk, int max_len, int window, int is_bf16) {
  if (window > 0 && max_len > window) max_len = window;
  if (!(is_bf16 && attn_latent_fits(k, d, dv, ldq, ldk, H))) return ell_attn_rows_scratch(n, H, 1, dv, max_len);
  const int s = attn_latent_splits(n, H, max_len);
  return s == 1 ? 0 : (long long)n * H * s * (dv + 2);
}

ELL_API int ell_attn_latent(const void* q, const void* k, void* out, float* part, const int* base, const int* len,
                            const void* gate, int n, int H, int d, int dv, int ldq, int ldk, int ldg, int max_len, int window,
                            long long rows, float scale, int is_bf16, int* err, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (!(is_bf16 && attn_latent_fits(k, d, dv, ldq, ldk, H)))
    return ell_attn_rows(q, k, k, out, part, base, len, nullptr, nullptr, gate, n, H, 1, d, dv, ldq, ldk, ldk, ldg, max_len,
                         window, scale, is_bf16, stream);
  if (!aligned_to(q, 16) || !aligned_to(k, 16) || !aligned_to(out, 16) || rows > 0x7fffffff) return -2;
  if (window <= 0) window = 0x7fffffff;
  if (max_len > window) max_len = window;
  AttnRowsArgs a{q, k, k, out, part, base, len, nullptr, nullptr, n, H, 1, d, dv, ldq, ldk, ldk, 1, 0, scale, window, gate, ldg, err};
  a.splits = attn_latent_splits(n, H, max_len);
  a.range = ((max_len + a.splits - 1) / a.splits + kAlKeys - 1) / kAlKeys * kAlKeys;
  if (a.splits > 1 && part == nullptr) return -2;
  return al_mt(H) == 1 ? launch_attn_latent<1>(a, rows, stream) : launch_attn_latent<2>(a, rows, stream);
}
