// Recurrent token mixers (inference): the short convolutions and gates of the gated delta rule, and the scans of the
// delta rule and of RWKV-style time mixing over packed sequences.  One source for prompts (long sequences) and decoding
// (one token); the recurrent state is fp32 throughout and so is everything that enters it.
//
// A state matrix S [d key rows x dv value columns] of one head evolves column by column without mixing columns:
//   time mixing   o_j = sum_i r_i (S_ij + u_i k_i v_j),          S_ij <- w_i S_ij + k_i v_j
//   delta rule    S_ij <- g_i S_ij,  e_j = beta (v_j - sum_i k_i S_ij),  S_ij <- S_ij + k_i e_j,  o_j = sum_i q_i S_ij
// so a CTA owns 32 columns of one (sequence, head) and no CTA waits for another.  A thread keeps 2 or 4 columns x 4 or
// 8 key rows in registers for the whole sequence (8 to 32 lanes share the columns): every operand word read from shared
// memory then serves several columns, which matters because filling registers from shared memory would otherwise limit
// a scan; with too many columns in a thread the latency of its chain does.  Both sums of the delta rule are taken from
// the decayed state at once (o_j = sum_i q_i g_i S_ij + (q . k) e_j), which leaves one shuffle reduction on the
// token-to-token chain; the sums of the thread's columns are reduced together, halving the number of values with every
// step.  Consumer warps run the recurrence on packed fp32 pairs (fma.rn.f32x2).  Eight more warps, one per token of a
// stage, copy the operands of the coming tokens into a ring of shared-memory stages with cp.async (three stages ahead),
// convert bf16 operands to fp32, compute the per-token scalars (q . k, or sum_i r_i u_i k_i), and write the previous
// tokens' outputs.
#include "vec.cuh"

namespace ell {

constexpr int kScanCols = 32;         // value columns of a CTA
constexpr int kScanTok = 8;           // tokens per stage
constexpr int kScanRing = 4;
constexpr int kLoadWarps = kScanTok;   // one token of a stage each

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

// packed pairs of fp32
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float sum2(f32x2 a) {
  float lo, hi;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(a));
  return lo + hi;
}

// One warp copies n <= N elements; vec: 16-byte pieces (start and length multiples of 16 bytes), else 4-byte ones (fp32).
template <typename T, int N>
__device__ __forceinline__ void warp_copy(T* dst, const T* src, int n, bool vec, int lane) {
  constexpr int kPer = 16 / sizeof(T);
  if (vec) {
#pragma unroll
    for (int b = 0; b < N; b += 32 * kPer) {
      const int c = b + lane * kPer;
      if (c < n) cp_async16(dst + c, src + c);
    }
  } else if (sizeof(T) == 4) {
    for (int c = lane; c < n; c += 32) cp_async4(dst + c, src + c);
  }
}

// Thread layout for heads of up to DP key rows (32, 64, 128 or 256): kLanes lanes hold the rows 4 l + 4 kLanes j .. + 3
// (j < kJ) of kCols columns.  Token record the recurrence reads: q | k | g | v | scalar, beta (fp32).  Raw bf16 record:
// g | beta (fp32), q | k | v.
template <int DP>
struct ScanTok {
  static constexpr int kLanes = DP <= 64 ? 8 : DP / 8;
  static constexpr int kJ = DP / (4 * kLanes);
  static constexpr int kCols = DP <= 128 ? 2 : 4;
  static constexpr int kWarpCols = kCols * (32 / kLanes);
  static constexpr int kWarps = kScanCols / kWarpCols;             // consumer warps
  static constexpr int kThreads = (kWarps + kLoadWarps) * 32;
  static constexpr int kFloats = 3 * DP + kScanCols + 4;
  static constexpr int kRawBytes = (DP + 4) * 4 + (2 * DP + kScanCols) * 2;
};
template <typename T, int DP>
__host__ __device__ constexpr int scan_smem_bytes() {
  using R = ScanTok<DP>;
  const int out = 2 * kScanTok * kScanCols * 4;
  return sizeof(T) == 4 ? kScanRing * kScanTok * R::kFloats * 4 + out
                        : 2 * kScanTok * R::kFloats * 4 + kScanRing * kScanTok * R::kRawBytes + out;
}

// Sums over the L lanes of a group of NV values per lane.  Each step halves the values a lane keeps (lanes with bit
// L / 2 set take the upper half, then L / 4, ...) until one is left, which is then summed over the remaining lanes.
template <int NV, int L>
__device__ __forceinline__ float reduce_columns(float* v, int l) {
  int n = NV;
#pragma unroll
  for (int o = L / 2; o >= 1; o >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool up = l & o;
#pragma unroll
      for (int i = 0; i < NV / 2; ++i) {
        if (i < n) {
          const float keep = up ? v[i + n] : v[i], give = up ? v[i] : v[i + n];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
      }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
    }
  }
  return v[0];
}

template <int MODE, typename T, int DP>
__global__ void __launch_bounds__(ScanTok<DP>::kThreads) scan_kernel(const ScanArgs a, int vec) {
  using R = ScanTok<DP>;
  constexpr int TF = R::kFloats, L = R::kLanes, J = R::kJ, NC = R::kCols;
  constexpr bool kF32 = sizeof(T) == 4;
  constexpr int kBufs = kF32 ? kScanRing : 2;          // fp32 records: the ring itself, or two converted stages
  extern __shared__ __align__(16) float sm[];
  float* outb = sm + kBufs * kScanTok * TF;            // [2][kScanTok][kScanCols]
  uint8_t* raw = reinterpret_cast<uint8_t*>(outb + 2 * kScanTok * kScanCols);
  const int s = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * kScanCols;
  const int t_begin = a.cu[s], n_tok = a.cu[s + 1] - t_begin;
  if (n_tok <= 0) return;
  const int hk = h / (a.H / a.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_chunk = (n_tok + kScanTok - 1) / kScanTok;
  const bool loader = warp >= R::kWarps;
  const int lw = warp - R::kWarps;                     // loader warp
  const int l = lane % L;                              // row slice
  const int cl = warp * R::kWarpCols + lane / L * NC;  // first of the thread's columns within the CTA

  // the copies never write past d and dv: what lies behind must read as zero
  for (int i = threadIdx.x; i < scan_smem_bytes<T, DP>() / 16; i += R::kThreads)
    reinterpret_cast<uint4*>(sm)[i] = make_uint4(0, 0, 0, 0);

  f32x2 S[NC][2 * J];                                  // [column][pair of rows]
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int i = 0; i < 2 * J; ++i) S[c][i] = 0ull;
  const int sp = (a.d + 31) / 32 * 32;                 // row stride of the stored state
  float* srow = nullptr;
  if (a.state != nullptr && !loader) {
    srow = a.state + (((size_t)a.slots[s] * a.H + h) * a.dv + col0 + cl) * sp + l * 4;
    if (a.pos0[s] > 0) {
#pragma unroll
      for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int j = 0; j < J; ++j)
          if (col0 + cl + c < a.dv && l * 4 + j * 4 * L < sp) {
            const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(srow + c * sp + j * 4 * L);
            S[c][2 * j] = x.x;
            S[c][2 * j + 1] = x.y;
          }
    }
  }
  __syncthreads();

  // loader warp lw owns token lw of every stage
  const size_t t_mine = (size_t)t_begin + lw;
  const T* q_src = reinterpret_cast<const T*>(a.q) + t_mine * a.ldq + (size_t)hk * a.d;
  const T* k_src = reinterpret_cast<const T*>(a.k) + t_mine * a.ldk + (size_t)hk * a.d;
  const T* v_src = reinterpret_cast<const T*>(a.v) + t_mine * a.ldv + (size_t)h * a.dv + col0;
  const float* g_src = a.g + (t_mine * a.H + h) * a.d;
  const float* b_src = MODE == kDelta ? a.beta + t_mine * a.H + h : nullptr;
  float* o_dst = a.o + (t_mine * a.H + h) * a.dv + col0 + lane;
  const size_t g_step = (size_t)kScanTok * a.H * a.d, o_step = (size_t)kScanTok * a.H * a.dv;
  const int nv = min(kScanCols, a.dv - col0);
  float u[DP / 32];                                    // wkv: the bonus of the loader lane's channels
#pragma unroll
  for (int c = 0; c < DP / 32; ++c)
    u[c] = MODE == kWkv && loader && c * 32 + lane < a.d ? a.u[(size_t)h * a.d + c * 32 + lane] : 0.f;

  auto issue = [&](int ch) {                           // start the copies of a stage
    if (ch * kScanTok + lw < n_tok) {
      float *gd, *bd;
      T *qd, *kd, *vd;
      if (kF32) {
        float* tok = sm + ((ch % kScanRing) * kScanTok + lw) * TF;
        qd = reinterpret_cast<T*>(tok), kd = qd + DP, gd = tok + 2 * DP, vd = reinterpret_cast<T*>(tok + 3 * DP);
        bd = tok + 3 * DP + kScanCols + 1;
      } else {
        uint8_t* rec = raw + ((ch % kScanRing) * kScanTok + lw) * R::kRawBytes;
        gd = reinterpret_cast<float*>(rec), bd = gd + DP, qd = reinterpret_cast<T*>(gd + DP + 4), kd = qd + DP, vd = kd + DP;
      }
      const size_t t = (size_t)ch * kScanTok;
      warp_copy<T, DP>(qd, q_src + t * a.ldq, a.d, vec, lane);
      warp_copy<T, DP>(kd, k_src + t * a.ldk, a.d, vec, lane);
      warp_copy<float, DP>(gd, g_src + ch * g_step, a.d, vec, lane);
      warp_copy<T, kScanCols>(vd, v_src + t * a.ldv, nv, vec, lane);
      if (MODE == kDelta && lane == 0) cp_async4(bd, b_src + t * a.H);
    }
    cp_async_commit();
  };
  auto prepare = [&](int ch) {                         // a landed stage: scalars, and fp32 records of bf16 operands
    cp_async_wait<kScanRing - 2>();
    __syncwarp();
    if (ch * kScanTok + lw >= n_tok) return;
    float* tok = sm + ((ch % kBufs) * kScanTok + lw) * TF;
    float dot = 0.f;
    if (kF32) {
#pragma unroll
      for (int c = 0; c < DP / 32; ++c) {
        const float p = tok[c * 32 + lane] * tok[DP + c * 32 + lane];
        dot = MODE == kWkv ? fmaf(p, u[c], dot) : dot + p;
      }
    } else {
      const float* gs = reinterpret_cast<const float*>(raw + ((ch % kScanRing) * kScanTok + lw) * R::kRawBytes);
      const size_t t = (size_t)ch * kScanTok;
      const T* qs = vec ? reinterpret_cast<const T*>(gs + DP + 4) : q_src + t * a.ldq;
      const T* ks = vec ? reinterpret_cast<const T*>(gs + DP + 4) + DP : k_src + t * a.ldk;
      const T* vs = vec ? reinterpret_cast<const T*>(gs + DP + 4) + 2 * DP : v_src + t * a.ldv;
#pragma unroll
      for (int c = 0; c < DP / 32; ++c) {
        const int x = c * 32 + lane;
        const bool in = x < a.d;
        const float q = in ? to_f<T>(qs[x]) : 0.f, k = in ? to_f<T>(ks[x]) : 0.f;
        tok[x] = q;
        tok[DP + x] = k;
        tok[2 * DP + x] = gs[x];
        dot = MODE == kWkv ? fmaf(q * k, u[c], dot) : fmaf(q, k, dot);
      }
      tok[3 * DP + lane] = lane < nv ? to_f<T>(vs[lane]) : 0.f;
      if (lane == 0) tok[3 * DP + kScanCols + 1] = gs[DP];
    }
    dot = warp_sum(dot);
    if (lane == 0) tok[3 * DP + kScanCols] = dot;
  };
  auto store = [&](int ch) {
    if (ch * kScanTok + lw < n_tok && lane < nv)
      o_dst[ch * o_step] = outb[((ch & 1) * kScanTok + lw) * kScanCols + lane];
  };

  if (loader) {
#pragma unroll
    for (int c = 0; c < kScanRing - 1; ++c) issue(c);
    prepare(0);
  }
  __syncthreads();
  for (int ch = 0; ch < n_chunk; ++ch) {
    if (loader) {
      issue(ch + kScanRing - 1);
      prepare(ch + 1);
      if (ch > 0) store(ch - 1);
    } else {
      const float* st = sm + (ch % kBufs) * kScanTok * TF;
      const int cnt = min(kScanTok, n_tok - ch * kScanTok);
      float* ob = outb + (ch & 1) * kScanTok * kScanCols;
      // after the reduction a lane holds the sum of one column (and, in the delta rule, of k or of q)
      constexpr int kTop = MODE == kDelta ? L / 4 : L / 2;            // lane bits: k or q | column, high bit first
      constexpr int kC0 = NC == 4 ? kTop / 2 : kTop, kC1 = NC == 4 ? kTop : 0;
      const int my_c = (l & kC1 ? 2 : 0) + (l & kC0 ? 1 : 0);
      const bool is_q = MODE == kWkv || (l & (L / 2));
      const bool writes = is_q && (l & (kC0 - 1)) == 0;
      float out[kScanTok];
      auto token = [&](int i) -> float {
        const float* tok = st + i * TF;
        const float sc = tok[3 * DP + kScanCols], v_mine = tok[3 * DP + cl + my_c];
        ulonglong2 q[J], k[J], g[J];
#pragma unroll
        for (int j = 0; j < J; ++j) {
          q[j] = *reinterpret_cast<const ulonglong2*>(tok + j * 4 * L + l * 4);
          k[j] = *reinterpret_cast<const ulonglong2*>(tok + DP + j * 4 * L + l * 4);
          g[j] = *reinterpret_cast<const ulonglong2*>(tok + 2 * DP + j * 4 * L + l * 4);
        }
        if (MODE == kWkv) {
          float sum[NC];
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            const float v = tok[3 * DP + cl + c];
            const f32x2 vv = pack2(v, v);
            f32x2 o = 0ull;
#pragma unroll
            for (int j = 0; j < J; ++j) {
              o = fma2(q[j].x, S[c][2 * j], o);
              o = fma2(q[j].y, S[c][2 * j + 1], o);
              S[c][2 * j] = fma2(g[j].x, S[c][2 * j], mul2(k[j].x, vv));
              S[c][2 * j + 1] = fma2(g[j].y, S[c][2 * j + 1], mul2(k[j].y, vv));
            }
            sum[c] = sum2(o);
          }
          return fmaf(sc, v_mine, reduce_columns<NC, L>(sum, l));
        } else {
          const float beta = tok[3 * DP + kScanCols + 1];
          float sum[2 * NC];
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            f32x2 ks = 0ull, qs = 0ull;
#pragma unroll
            for (int j = 0; j < J; ++j) {
              S[c][2 * j] = mul2(S[c][2 * j], g[j].x);
              S[c][2 * j + 1] = mul2(S[c][2 * j + 1], g[j].y);
              ks = fma2(k[j].x, S[c][2 * j], ks);
              qs = fma2(q[j].x, S[c][2 * j], qs);
              ks = fma2(k[j].y, S[c][2 * j + 1], ks);
              qs = fma2(q[j].y, S[c][2 * j + 1], qs);
            }
            sum[c] = sum2(ks);
            sum[NC + c] = sum2(qs);
          }
          const float mine = reduce_columns<2 * NC, L>(sum, l);
          const float e = beta * (v_mine - mine);      // of the lanes that hold a k sum
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            const float ec = __shfl_sync(0xffffffffu, e, (lane & ~(L - 1)) + (c & 2 ? kC1 : 0) + (c & 1 ? kC0 : 0));
            const f32x2 ee = pack2(ec, ec);
#pragma unroll
            for (int j = 0; j < J; ++j) {
              S[c][2 * j] = fma2(k[j].x, ee, S[c][2 * j]);
              S[c][2 * j + 1] = fma2(k[j].y, ee, S[c][2 * j + 1]);
            }
          }
          return fmaf(sc, __shfl_xor_sync(0xffffffffu, e, L / 2), mine);
        }
      };
      if (cnt == kScanTok) {
#pragma unroll
        for (int i = 0; i < kScanTok; ++i) out[i] = token(i);
#pragma unroll
        for (int i = 0; i < kScanTok; ++i)
          if (writes) ob[i * kScanCols + cl + my_c] = out[i];
      } else {
        for (int i = 0; i < cnt; ++i) {
          const float o = token(i);
          if (writes) ob[i * kScanCols + cl + my_c] = o;
        }
      }
    }
    __syncthreads();
  }
  if (loader) {
    store(n_chunk - 1);
  } else if (srow != nullptr) {
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int j = 0; j < J; ++j)
        if (col0 + cl + c < a.dv && l * 4 + j * 4 * L < sp)
          *reinterpret_cast<ulonglong2*>(srow + c * sp + j * 4 * L) = make_ulonglong2(S[c][2 * j], S[c][2 * j + 1]);
  }
}

template <int MODE, typename T, int DP>
int launch_scan(const ScanArgs& a, int n_seq, int vec, cudaStream_t stream) {
  constexpr int bytes = scan_smem_bytes<T, DP>();
  auto kern = scan_kernel<MODE, T, DP>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  dim3 grid((a.dv + kScanCols - 1) / kScanCols, a.H, n_seq);
  kern<<<grid, ScanTok<DP>::kThreads, bytes, stream>>>(a, vec);
  return launch_status();
}

template <int MODE, typename T>
int dispatch_scan(const ScanArgs& a, int n_seq, cudaStream_t stream) {
  // 16-byte copies: every head starts on a 16-byte boundary and is a multiple of 16 bytes long
  constexpr int per = 16 / sizeof(T);
  const int v = a.d % per == 0 && a.dv % per == 0 && a.d % 4 == 0 && a.ldq % per == 0 && a.ldk % per == 0 &&
                a.ldv % per == 0 && aligned_to(a.q, 16) && aligned_to(a.k, 16) && aligned_to(a.v, 16) && aligned_to(a.g, 16);
  if (a.d <= 32) return launch_scan<MODE, T, 32>(a, n_seq, v, stream);
  if (a.d <= 64) return launch_scan<MODE, T, 64>(a, n_seq, v, stream);
  if (a.d <= 128) return launch_scan<MODE, T, 128>(a, n_seq, v, stream);
  if (a.d <= 256) return launch_scan<MODE, T, 256>(a, n_seq, v, stream);
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

// Sums over the 32 lanes of 16 values per lane: lane l returns the total of value l >> 1.
__device__ __forceinline__ float warp_sum16(float* v) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 16, n = 8; o >= 2; o >>= 1, n >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (i < n) {
        const float keep = up ? v[i + n] : v[i], give = up ? v[i] : v[i + n];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
      }
    }
  }
  return v[0] + __shfl_xor_sync(0xffffffffu, v[0], 1);
}

// blockIdx.x: a q head, a k head, a v head, or the decays of a head; blockIdx.y: chunk of tokens; blockIdx.z: sequence.
// Thread c is channel c of the head.  Only chunk 0 reaches in front of the sequence, so it alone reads the tail, and
// it replaces it by the sequence's last inputs afterwards (each thread its own channel).  NT: taps (0: any number).
template <typename T, int NT>
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
    float z[kConvTok];
    if (c < p.d) {
      float* base = p.a + head * p.d + c;
#pragma unroll
      for (int i = 0; i < kConvTok; ++i) z[i] = base[(size_t)min(t0 + i, t1 - 1) * p.H * p.d];
      const float dt = p.dt_bias[head * p.d + c];
#pragma unroll
      for (int i = 0; i < kConvTok; ++i)
        if (t0 + i < t1) base[(size_t)(t0 + i) * p.H * p.d] = expf(-rate * softplus_f(z[i] + dt));
    }
    if (c < t1 - t0) p.beta[(size_t)(t0 + c) * p.H + head] = sigmoid_f(p.b[(size_t)(t0 + c) * p.ldb + head]);
    return;
  }
  const bool is_v = head >= 2 * p.G;
  const int width = is_v ? p.dv : p.d;
  const int n_taps = NT > 0 ? NT : p.n_taps;
  const int C = 2 * p.G * p.d + p.H * p.dv, n1 = n_taps - 1;
  const int ch = is_v ? 2 * p.G * p.d + (head - 2 * p.G) * p.dv + c : head * p.d + c;
  const T* x = reinterpret_cast<const T*>(p.x) + ch;
  float y[kConvTok];
#pragma unroll
  for (int i = 0; i < kConvTok; ++i) y[i] = 0.f;
  if (c < width) {
    T* tail = p.tail != nullptr ? reinterpret_cast<T*>(p.tail) + ((size_t)p.slots[s] * C + ch) * n1 : nullptr;
    const bool past = tail != nullptr && p.pos0[s] > 0;
    constexpr int kReach = NT > 0 ? NT - 1 : kConvTok;
    float w[kReach + kConvTok];                           // inputs t0 - kReach .. t0 + 15
    if (t0 - kReach >= sa) {                              // the usual case: all loads at once, no branches
      const T* xp = x + (size_t)(t0 - kReach) * p.ldx;
      T raw[kReach + kConvTok];
#pragma unroll
      for (int i = 0; i < kReach + kConvTok; ++i) raw[i] = xp[(size_t)min(i, t1 - 1 - t0 + kReach) * p.ldx];
#pragma unroll
      for (int i = 0; i < kReach + kConvTok; ++i) w[i] = to_f<T>(raw[i]);
    } else {
#pragma unroll
      for (int i = 0; i < kReach + kConvTok; ++i) {
        const int t = t0 - kReach + i;
        w[i] = 0.f;
        if (t >= sa) w[i] = to_f<T>(x[(size_t)min(t, t1 - 1) * p.ldx]);
        else if (past && t >= sa - n1) w[i] = to_f<T>(tail[n1 + t - sa]);
      }
    }
#pragma unroll
    for (int j = 0; j <= kReach; ++j) {                   // tap of the input j tokens back
      if (j <= n1) {
        const float tap = p.taps[(size_t)ch * n_taps + n1 - j];
#pragma unroll
        for (int i = 0; i < kConvTok; ++i) y[i] = fmaf(tap, w[kReach + i - j], y[i]);
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
    if (c < width) {
      float* out = p.v + (size_t)(head - 2 * p.G) * p.dv + c;
#pragma unroll
      for (int i = 0; i < kConvTok; ++i)
        if (t0 + i < t1) out[(size_t)(t0 + i) * p.H * p.dv] = y[i];
    }
    return;
  }
  float sq[kConvTok];
#pragma unroll
  for (int i = 0; i < kConvTok; ++i) sq[i] = y[i] * y[i];
  const float ss = warp_sum16(sq);
  if (!(lane & 1)) red[lane >> 1][warp] = ss;
  __syncthreads();
  const bool is_q = head < p.G;
  float* out = (is_q ? p.q : p.k) + (size_t)(is_q ? head : head - p.G) * p.d + c;
  const float mul = is_q ? 1.f / sqrtf((float)p.d) : 1.f;
  if (threadIdx.x < kConvTok) {
    float t = 0.f;
    for (int w = 0; w < nw; ++w) t += red[threadIdx.x][w];
    red[threadIdx.x][32] = mul / sqrtf(t + 1e-6f);
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < kConvTok; ++i)
    if (t0 + i < t1 && c < width) out[(size_t)(t0 + i) * p.G * p.d] = y[i] * red[i][32];
}

template <typename T>
static void launch_delta_inputs(const DeltaInArgs& p, dim3 grid, int threads, cudaStream_t stream) {
  switch (p.n_taps) {
    case 1: delta_inputs_kernel<T, 1><<<grid, threads, 0, stream>>>(p); break;
    case 2: delta_inputs_kernel<T, 2><<<grid, threads, 0, stream>>>(p); break;
    case 3: delta_inputs_kernel<T, 3><<<grid, threads, 0, stream>>>(p); break;
    case 4: delta_inputs_kernel<T, 4><<<grid, threads, 0, stream>>>(p); break;
    default: delta_inputs_kernel<T, 0><<<grid, threads, 0, stream>>>(p);
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
  if (is_bf16) launch_delta_inputs<__nv_bfloat16>(p, grid, threads, stream);
  else launch_delta_inputs<float>(p, grid, threads, stream);
  return launch_status();
}
