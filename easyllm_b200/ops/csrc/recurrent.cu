// Recurrent token mixers (inference): the short convolutions and gates of the gated delta rule, and the scans of the
// delta rule and of RWKV-style time mixing over packed sequences.  One source for prompts (long sequences) and decoding
// (one token); the recurrent state is fp32 throughout and so is everything that enters it.
//
// A state matrix S [d key rows x dv value columns] of one head evolves column by column without mixing columns:
//   time mixing   o_j = sum_i r_i (S_ij + u_i k_i v_j),          S_ij <- w_i S_ij + k_i v_j
//   delta rule    S_ij <- g_i S_ij,  e_j = beta (v_j - sum_i k_i S_ij),  S_ij <- S_ij + k_i e_j,  o_j = sum_i q_i S_ij
// so a CTA owns 32 columns of one (sequence, head) and no CTA waits for another.  Eight lanes share a column: lane r
// keeps rows 32 i + 4 r .. + 3 in registers for the whole sequence.  Both sums of the delta rule are taken from the
// decayed state at once (o_j = sum_i q_i g_i S_ij + (q . k) e_j), which leaves one shuffle reduction on the
// token-to-token chain.
// Warps 0-7 run the recurrence; warps 8-11 stage the next tokens' operands in shared memory (two buffers), compute the
// per-token scalars (q . k, or sum_i r_i u_i k_i), and write the previous tokens' outputs.
#include "vec.cuh"

namespace ell {

constexpr int kScanCols = 32;         // value columns of a CTA
constexpr int kScanTok = 16;          // tokens per stage
constexpr int kScanWarps = 8, kLoadWarps = 4;
constexpr int kScanThreads = (kScanWarps + kLoadWarps) * 32;

enum ScanMode { kWkv = 0, kDelta = 1 };

struct ScanArgs {
  const void *q, *k, *v;        // delta: fp32; wkv: activation type.  q is r in wkv
  const float *g;               // decay [n, H, d]
  const float *beta;            // delta: [n, H]
  const float *u;               // wkv: [H, d]
  float* o;                     // [n, H, dv]
  float* state;                 // [slots, H, dv, dp] or null
  const int *cu, *slots, *pos0;
  int H, G, d, dv, ldq, ldk, ldv;   // row strides of q, k, v in elements
};

template <typename T>
__device__ __forceinline__ float4 load4_guard(const T* p, int c, int d, bool vec) {
  float f[4] = {0.f, 0.f, 0.f, 0.f};
  if (vec && c + 3 < d) {
    load_v<4>(p + c, f);
  } else {
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (c + j < d) f[j] = to_f<T>(p[c + j]);
  }
  return make_float4(f[0], f[1], f[2], f[3]);
}

template <int MODE, typename T, int NI>
__global__ void __launch_bounds__(kScanThreads) scan_kernel(const ScanArgs a, int vec) {
  constexpr int DP = NI * 32;
  constexpr int kTokFloats = 3 * DP + kScanCols + 4;   // q | k | g | v | scalar, beta
  extern __shared__ float sm[];
  float* stage[2] = {sm, sm + kScanTok * kTokFloats};
  float* outb = sm + 2 * kScanTok * kTokFloats;        // [2][kScanTok][kScanCols]
  const int s = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * kScanCols;
  const int t_begin = a.cu[s], n_tok = a.cu[s + 1] - t_begin;
  if (n_tok <= 0) return;
  const int hk = h / (a.H / a.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_chunk = (n_tok + kScanTok - 1) / kScanTok;
  const bool loader = warp >= kScanWarps;
  const int r = lane & 7;
  const int cl = (warp & 7) * 4 + (lane >> 3);         // column within the CTA
  const int col = col0 + cl;
  const bool live = !loader && col < a.dv;

  auto load_chunk = [&](int ch) {
    float* st = stage[ch & 1];
    const int cnt = min(kScanTok, n_tok - ch * kScanTok);
    for (int i = warp - kScanWarps; i < cnt; i += kLoadWarps) {
      const size_t t = (size_t)t_begin + ch * kScanTok + i;
      float* tok = st + i * kTokFloats;
      const T* qp = reinterpret_cast<const T*>(a.q) + t * a.ldq + (size_t)hk * a.d;
      const T* kp = reinterpret_cast<const T*>(a.k) + t * a.ldk + (size_t)hk * a.d;
      const float* gp = a.g + (t * a.H + h) * a.d;
      float dot = 0.f;
#pragma unroll
      for (int c0 = 0; c0 < DP; c0 += 128) {
        const int c = c0 + lane * 4;
        if (c < DP) {
          const float4 q = load4_guard<T>(qp, c, a.d, vec), k = load4_guard<T>(kp, c, a.d, vec);
          const float4 g = load4_guard<float>(gp, c, a.d, vec);
          *reinterpret_cast<float4*>(tok + c) = q;
          *reinterpret_cast<float4*>(tok + DP + c) = k;
          *reinterpret_cast<float4*>(tok + 2 * DP + c) = g;
          if (MODE == kWkv) {
            const float4 u = load4_guard<float>(a.u + (size_t)h * a.d, c, a.d, vec);
            dot += q.x * k.x * u.x + q.y * k.y * u.y + q.z * k.z * u.z + q.w * k.w * u.w;
          } else {
            dot += q.x * k.x + q.y * k.y + q.z * k.z + q.w * k.w;
          }
        }
      }
      const int c = col0 + lane;
      tok[3 * DP + lane] = c < a.dv ? to_f<T>(reinterpret_cast<const T*>(a.v)[t * a.ldv + (size_t)h * a.dv + c]) : 0.f;
      dot = warp_sum(dot);
      if (lane == 0) {
        tok[3 * DP + kScanCols] = dot;
        if (MODE == kDelta) tok[3 * DP + kScanCols + 1] = a.beta[t * a.H + h];
      }
    }
  };
  auto store_chunk = [&](int ch) {
    const float* ob = outb + (ch & 1) * kScanTok * kScanCols;
    const int cnt = min(kScanTok, n_tok - ch * kScanTok);
    for (int i = warp - kScanWarps; i < cnt; i += kLoadWarps) {
      const size_t t = (size_t)t_begin + ch * kScanTok + i;
      if (col0 + lane < a.dv) a.o[(t * a.H + h) * a.dv + col0 + lane] = ob[i * kScanCols + lane];
    }
  };

  float S[4 * NI];
#pragma unroll
  for (int i = 0; i < 4 * NI; ++i) S[i] = 0.f;
  float* srow = nullptr;
  if (a.state != nullptr && live) {
    srow = a.state + (((size_t)a.slots[s] * a.H + h) * a.dv + col) * DP + r * 4;
    if (a.pos0[s] > 0) {
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float4 x = *reinterpret_cast<const float4*>(srow + i * 32);
        S[4 * i] = x.x; S[4 * i + 1] = x.y; S[4 * i + 2] = x.z; S[4 * i + 3] = x.w;
      }
    }
  }
  if (loader) load_chunk(0);
  __syncthreads();
  for (int ch = 0; ch < n_chunk; ++ch) {
    if (loader) {
      if (ch + 1 < n_chunk) load_chunk(ch + 1);
      if (ch > 0) store_chunk(ch - 1);
    } else {
      const float* st = stage[ch & 1];
      float* ob = outb + (ch & 1) * kScanTok * kScanCols;
      const int cnt = min(kScanTok, n_tok - ch * kScanTok);
      for (int i = 0; i < cnt; ++i) {
        const float* tok = st + i * kTokFloats;
        const float v = tok[3 * DP + cl], sc = tok[3 * DP + kScanCols];
        if (MODE == kWkv) {
          float o0 = 0.f, o1 = 0.f;
#pragma unroll
          for (int j = 0; j < NI; ++j) {
            const float4 q = *reinterpret_cast<const float4*>(tok + j * 32 + r * 4);
            const float4 k = *reinterpret_cast<const float4*>(tok + DP + j * 32 + r * 4);
            const float4 g = *reinterpret_cast<const float4*>(tok + 2 * DP + j * 32 + r * 4);
            float* x = S + 4 * j;
            o0 = fmaf(q.x, x[0], o0); o1 = fmaf(q.y, x[1], o1);
            o0 = fmaf(q.z, x[2], o0); o1 = fmaf(q.w, x[3], o1);
            x[0] = fmaf(g.x, x[0], k.x * v); x[1] = fmaf(g.y, x[1], k.y * v);
            x[2] = fmaf(g.z, x[2], k.z * v); x[3] = fmaf(g.w, x[3], k.w * v);
          }
          float o = o0 + o1;
          o += __shfl_xor_sync(0xffffffffu, o, 1);
          o += __shfl_xor_sync(0xffffffffu, o, 2);
          o += __shfl_xor_sync(0xffffffffu, o, 4);
          if (r == 0) ob[i * kScanCols + cl] = fmaf(sc, v, o);
        } else {
          const float beta = tok[3 * DP + kScanCols + 1];
          float k0 = 0.f, k1 = 0.f, q0 = 0.f, q1 = 0.f;
          float kk[4 * NI];
#pragma unroll
          for (int j = 0; j < NI; ++j) {
            const float4 q = *reinterpret_cast<const float4*>(tok + j * 32 + r * 4);
            const float4 k = *reinterpret_cast<const float4*>(tok + DP + j * 32 + r * 4);
            const float4 g = *reinterpret_cast<const float4*>(tok + 2 * DP + j * 32 + r * 4);
            float* x = S + 4 * j;
            kk[4 * j] = k.x; kk[4 * j + 1] = k.y; kk[4 * j + 2] = k.z; kk[4 * j + 3] = k.w;
            x[0] *= g.x; x[1] *= g.y; x[2] *= g.z; x[3] *= g.w;
            k0 = fmaf(k.x, x[0], k0); k1 = fmaf(k.y, x[1], k1);
            q0 = fmaf(q.x, x[0], q0); q1 = fmaf(q.y, x[1], q1);
            k0 = fmaf(k.z, x[2], k0); k1 = fmaf(k.w, x[3], k1);
            q0 = fmaf(q.z, x[2], q0); q1 = fmaf(q.w, x[3], q1);
          }
          // even lanes reduce the k sum, odd lanes the q sum
          const float ks = k0 + k1, qs = q0 + q1;
          float mine = (r & 1) ? qs : ks;
          mine += __shfl_xor_sync(0xffffffffu, (r & 1) ? ks : qs, 1);
          mine += __shfl_xor_sync(0xffffffffu, mine, 2);
          mine += __shfl_xor_sync(0xffffffffu, mine, 4);
          const float other = __shfl_xor_sync(0xffffffffu, mine, 1);
          const float e = beta * (v - ((r & 1) ? other : mine));
          if (r == 0) ob[i * kScanCols + cl] = fmaf(sc, e, other);
#pragma unroll
          for (int j = 0; j < 4 * NI; ++j) S[j] = fmaf(kk[j], e, S[j]);
        }
      }
    }
    __syncthreads();
  }
  if (loader) {
    store_chunk(n_chunk - 1);
  } else if (srow != nullptr) {
#pragma unroll
    for (int i = 0; i < NI; ++i)
      *reinterpret_cast<float4*>(srow + i * 32) = make_float4(S[4 * i], S[4 * i + 1], S[4 * i + 2], S[4 * i + 3]);
  }
}

template <int MODE, typename T, int NI>
int launch_scan(const ScanArgs& a, int n_seq, int vec, cudaStream_t stream) {
  constexpr int bytes = (2 * kScanTok * (3 * NI * 32 + kScanCols + 4) + 2 * kScanTok * kScanCols) * 4;
  auto kern = scan_kernel<MODE, T, NI>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  dim3 grid((a.dv + kScanCols - 1) / kScanCols, a.H, n_seq);
  kern<<<grid, kScanThreads, bytes, stream>>>(a, vec);
  return launch_status();
}

template <int MODE, typename T>
int dispatch_scan(const ScanArgs& a, int n_seq, cudaStream_t stream) {
  const int v = a.d % 4 == 0 && a.ldq % 4 == 0 && a.ldk % 4 == 0 && aligned_to(a.q, 16) && aligned_to(a.k, 16) &&
                aligned_to(a.g, 16) && aligned_to(a.u, 16);
  switch ((a.d + 31) / 32) {
    case 1: return launch_scan<MODE, T, 1>(a, n_seq, v, stream);
    case 2: return launch_scan<MODE, T, 2>(a, n_seq, v, stream);
    case 3: return launch_scan<MODE, T, 3>(a, n_seq, v, stream);
    case 4: return launch_scan<MODE, T, 4>(a, n_seq, v, stream);
    case 5: return launch_scan<MODE, T, 5>(a, n_seq, v, stream);
    case 6: return launch_scan<MODE, T, 6>(a, n_seq, v, stream);
    case 7: return launch_scan<MODE, T, 7>(a, n_seq, v, stream);
    case 8: return launch_scan<MODE, T, 8>(a, n_seq, v, stream);
  }
  return -2;
}

// ---- inputs of the delta rule -------------------------------------------------------------------
constexpr int kConvTok = 16;          // tokens a block walks; the number of taps is at most kConvTok + 1

struct DeltaInArgs {
  const void* x;                // [n, C] projections, C = 2 G d + H dv (q | k | v), rows of ldx
  const float* taps;            // [C, n_taps]
  float* a;                     // [n, H d] in: decay logits, out: decays
  const float *A_log, *dt_bias; // [H], [H d]
  const float* b;               // [n, H] step-size logits, rows of ldb
  float *q, *k, *v, *beta;      // out
  void* tail;                   // [slots, C, n_taps - 1], oldest first, or null
  const int *cu, *slots, *pos0;
  int H, G, d, dv, n_taps, ldx, ldb;
};

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// blockIdx.x: a q head, a k head, a v head, or the decays of a head; blockIdx.y: chunk of tokens; blockIdx.z: sequence.
// Thread c is channel c of the head.  Only chunk 0 reaches in front of the sequence, so it alone reads the tail, and
// it replaces it by the sequence's last inputs afterwards (each thread its own channel).
template <typename T>
__global__ void delta_inputs_kernel(const DeltaInArgs p) {
  __shared__ float red[kConvTok][33];
  const int s = blockIdx.z, sa = p.cu[s], sb = p.cu[s + 1];
  const int t0 = sa + blockIdx.y * kConvTok, t1 = min(t0 + kConvTok, sb);
  if (t0 >= t1) return;
  const int c = threadIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  int head = blockIdx.x;
  if (head >= 2 * p.G + p.H) {
    head -= 2 * p.G + p.H;
    const float rate = expf(p.A_log[head]);
    for (int t = t0; t < t1; ++t) {
      if (c < p.d) {
        float* z = p.a + (size_t)t * p.H * p.d + head * p.d + c;
        *z = expf(-rate * softplus_f(*z + p.dt_bias[head * p.d + c]));
      }
      if (c == 0) p.beta[(size_t)t * p.H + head] = sigmoid_f(p.b[(size_t)t * p.ldb + head]);
    }
    return;
  }
  const bool is_v = head >= 2 * p.G;
  const int width = is_v ? p.dv : p.d;
  const int C = 2 * p.G * p.d + p.H * p.dv, n1 = p.n_taps - 1;
  const int ch = is_v ? 2 * p.G * p.d + (head - 2 * p.G) * p.dv + c : head * p.d + c;
  const T* x = reinterpret_cast<const T*>(p.x) + ch;
  float y[kConvTok];
#pragma unroll
  for (int i = 0; i < kConvTok; ++i) y[i] = 0.f;
  if (c < width) {
    T* tail = p.tail != nullptr ? reinterpret_cast<T*>(p.tail) + ((size_t)p.slots[s] * C + ch) * n1 : nullptr;
    const bool past = tail != nullptr && p.pos0[s] > 0;
    for (int j = 0; j <= n1; ++j) {                       // tap of the input j tokens back
      const float w = p.taps[(size_t)ch * p.n_taps + n1 - j];
#pragma unroll
      for (int i = 0; i < kConvTok; ++i) {
        const int t = t0 + i - j;
        if (t0 + i < t1) {
          if (t >= sa) y[i] = fmaf(w, to_f<T>(x[(size_t)t * p.ldx]), y[i]);
          else if (past) y[i] = fmaf(w, to_f<T>(tail[n1 + t - sa]), y[i]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < kConvTok; ++i) y[i] = silu_f(y[i]);
    if (tail != nullptr && blockIdx.y == 0) {
      const int len = sb - sa;
      for (int i = 0; i < n1; ++i) {                      // ascending: entry i + len is read before it is replaced
        const int t = len - n1 + i;                       // token of the sequence, negative: in the old tail
        tail[i] = t >= 0 ? x[(size_t)(sa + t) * p.ldx] : (past ? tail[n1 + t] : from_f<T>(0.f));
      }
    }
  }
  if (is_v) {
    if (c < width)
      for (int i = 0; t0 + i < t1; ++i) p.v[((size_t)(t0 + i) * p.H + head - 2 * p.G) * p.dv + c] = y[i];
    return;
  }
#pragma unroll
  for (int i = 0; i < kConvTok; ++i) {
    const float ss = warp_sum(y[i] * y[i]);
    if (lane == 0) red[i][warp] = ss;
  }
  __syncthreads();
  const bool is_q = head < p.G;
  float* out = (is_q ? p.q : p.k) + (size_t)(is_q ? head : head - p.G) * p.d + c;
  const float mul = is_q ? 1.f / sqrtf((float)p.d) : 1.f;
#pragma unroll
  for (int i = 0; i < kConvTok; ++i) {
    if (t0 + i < t1 && c < width) {
      float ss = 0.f;
      for (int w = 0; w < nw; ++w) ss += red[i][w];
      out[(size_t)(t0 + i) * p.G * p.d] = y[i] / sqrtf(ss + 1e-6f) * mul;
    }
  }
}

}  // namespace ell

using namespace ell;

// RWKV-style scan.  r, k, v: rows of ldr / ldk / ldv elements of the activation type; decay fp32 [n, H, d]; u [H, d].
ELL_API int ell_wkv_scan(const void* r, const void* k, const void* v, const float* decay, const float* u, float* o,
                         float* state, const int* cu, const int* slots, const int* pos0, int n_seq, int H, int d, int dv,
                         int ldr, int ldk, int ldv, int is_bf16, cudaStream_t stream) {
  if (n_seq <= 0) return 0;
  if (n_seq > 65535 || H > 65535) return -2;
  ScanArgs a{r, k, v, decay, nullptr, u, o, state, cu, slots, pos0, H, H, d, dv, ldr, ldk, ldv};
  return is_bf16 ? dispatch_scan<kWkv, __nv_bfloat16>(a, n_seq, stream) : dispatch_scan<kWkv, float>(a, n_seq, stream);
}

// Gated delta rule.  q, k fp32 [n, G, d], v fp32 [n, H, dv], decay fp32 [n, H, d], beta fp32 [n, H].
ELL_API int ell_delta_scan(const float* q, const float* k, const float* v, const float* decay, const float* beta, float* o,
                           float* state, const int* cu, const int* slots, const int* pos0, int n_seq, int H, int G, int d,
                           int dv, cudaStream_t stream) {
  if (n_seq <= 0) return 0;
  if (H % G || n_seq > 65535 || H > 65535) return -2;
  ScanArgs a{q, k, v, decay, beta, nullptr, o, state, cu, slots, pos0, H, G, d, dv, G * d, G * d, H * dv};
  return dispatch_scan<kDelta, float>(a, n_seq, stream);
}

ELL_API int ell_delta_inputs(const void* x, const float* taps, float* a, const float* A_log, const float* dt_bias,
                             const float* b, float* q, float* k, float* v, float* beta, void* tail, const int* cu,
                             const int* slots, const int* pos0, int n_seq, int max_len, int H, int G, int d, int dv,
                             int n_taps, int ldx, int ldb, int is_bf16, cudaStream_t stream) {
  if (n_seq <= 0 || max_len <= 0) return 0;
  const int width = d > dv ? d : dv, chunks = (max_len + kConvTok - 1) / kConvTok;
  if (n_taps < 1 || n_taps > kConvTok + 1 || width > 1024 || n_seq > 65535 || chunks > 65535) return -2;
  DeltaInArgs p{x, taps, a, A_log, dt_bias, b, q, k, v, beta, tail, cu, slots, pos0, H, G, d, dv, n_taps, ldx, ldb};
  dim3 grid(2 * G + 2 * H, chunks, n_seq);
  const int threads = (width + 31) / 32 * 32;
  if (is_bf16) delta_inputs_kernel<__nv_bfloat16><<<grid, threads, 0, stream>>>(p);
  else delta_inputs_kernel<float><<<grid, threads, 0, stream>>>(p);
  return launch_status();
}
