// Gated linear attention (sm_100a, float32 throughout): per request and head a state S [dk, dv] with a decay per key
// channel,
//
//   S_t = diag(exp(l_t)) S_(t-1) + k_t v_t^T,   o_t = S_t^T (q_scale q_t),
//   l_t = log sigmoid(A_2 a_t + b) / tau         (a_t: the first step of the decay's low-rank projection),
//   out_t = o_t / rms(o_t) * w * act(g_t)        per head; act = SiLU or sigmoid.
//
// Two ways to the same numbers, chosen by the longest run of tokens a request brings:
//
//   * gla_few_kernel (decoding, portions of a few tokens): a CTA per (request, head) holds S in registers and takes the
//     tokens one by one.  S changes by (exp(l) - 1) S + k v^T, the bracket by expm1: a decay near 1, rounded to float32,
//     would forget a few per cent faster or slower, always to the same side.
//   * chunks of 64 tokens (prompt portions), counted from a request's first token of the step:
//       gla_decay_kernel        l of every token and channel;
//       gla_chunk_state_kernel  per (chunk, head): sum_s (k_s exp(l_(s+1) + .. + l_end)) v_s^T, and the chunk's decay;
//       gla_state_scan_kernel   over a request's chunks: the state every chunk starts from; the last one is stored;
//       gla_chunk_out_kernel    per (chunk, head): with P_t = l_1 + .. + l_t inside the chunk
//                               o_t = (q_t exp(P_t)) S_start + sum_{s <= t} (sum_d q_td k_sd exp(P_td - P_sd)) v_s,
//                               then the norm, the weight and the gate.
//     The inner sums factor as (q exp(P)) (k exp(-P)) while no channel of a slice of 32 decays by more than exp(-30)
//     over the chunk, so that neither factor leaves float32's range; a slice that does takes running products of the
//     decays instead, which are exact for any decay.  All other exponents are sums of l over tokens that lie BEHIND the
//     one they weigh, hence <= 0.
//
// A row's order of additions is fixed by its place in its request's run, not by what else the step holds.
#include "linear_attention.cuh"

namespace {

constexpr int CH = 64;            // tokens per chunk
constexpr int TP = CH + 4;        // pitch of a [channel][token] tile that is read four tokens at a time
constexpr int SP = CH + 1;        // pitch of a [channel][token] tile that is read token by token
constexpr int SL = 32;            // channels per slice of the output kernel
constexpr int VT = 128;           // value channels per tile
constexpr float FACTOR_LIMIT = 30.f;

struct GlaArgs {
  const float* q; long ldq; const float* k; long ldk; const float* v; long ldv; const float* g; long ldg;
  const float* a1; long lda; const void* a2; int a2_dtype; const void* a2b; int b_dtype; int rank; float inv_tau;
  float q_scale;
  float* state; long state_stride;
  const int* cu_q; const int* state_slots;
  const void* norm_w; int norm_dtype; float eps; int gate_act;
  void* out; int out_dtype; long ldo;
  float* log_decay;       // [T][H dk]
  float* chunk_state;     // [T / CH + B][H][dk][dv]: request r's chunk c is row cu_q[r] / CH + r + c
  float* chunk_decay;     // [T / CH + B][H][dk]
  float* o_raw;           // [T][H dv], used when dv > VT
  int T, B, H, dk, dv;
};

__device__ __forceinline__ float gla_log_decay(float z, float inv_tau) {
  return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau;
}
__device__ __forceinline__ void gla_store(const GlaArgs& A, size_t t, size_t col, float x) {
  if (A.out_dtype == CO_BF16) ((__nv_bfloat16*)A.out)[t * A.ldo + col] = __float2bfloat16_rn(x);
  else ((float*)A.out)[t * A.ldo + col] = x;
}
// ------------------------------------------------------------------------------------------- few tokens per request
// grid (H, B), 256 threads.  Thread (warp y, lane x) owns rows y, y + 8, .. of S and four neighbouring columns of a tile of
// 128.  ROWS: rows a thread keeps in registers (0: the state stays in memory, for dk > 256).
// smem: q, k, exp(l) - 1 [L][dk] each, v, o [L][dv] each, partial sums [8][VT]; L = tokens of the longest run.
template <int ROWS>
__global__ void __launch_bounds__(256) gla_few_kernel(GlaArgs A, int L, bool vec) {
  extern __shared__ __align__(16) float sm[];
  co_pdl_launch_dependents();
  const int h = blockIdx.x, b = blockIdx.y, dk = A.dk, dv = A.dv;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* part = sm;                     // [8][VT]
  float* qs = part + 8 * VT;
  float* ks = qs + L * dk;
  float* es = ks + L * dk;
  float* vs = es + L * dk;
  float* os = vs + L * dv;
  co_pdl_wait();
  const int t0 = A.cu_q[b], n = A.cu_q[b + 1] - t0;
  if (n <= 0) return;
  float* S = A.state + (size_t)A.state_slots[b] * A.state_stride + (size_t)h * dk * dv;
  for (int e = threadIdx.x; e < n * dk; e += blockDim.x) {
    const int t = e / dk, c = e - t * dk;
    const size_t row = t0 + t;
    const size_t ch = (size_t)h * dk + c;
    qs[e] = A.q[row * A.ldq + ch] * A.q_scale;
    ks[e] = A.k[row * A.ldk + ch];
    float z = A.a2b ? co_load_any(A.a2b, A.b_dtype, ch) : 0.f;
    for (int r = 0; r < A.rank; ++r) z = fmaf(co_load_any(A.a2, A.a2_dtype, ch * A.rank + r), A.a1[row * A.lda + r], z);
    es[e] = expm1f(gla_log_decay(z, A.inv_tau));
  }
  for (int e = threadIdx.x; e < n * dv; e += blockDim.x) {
    const int t = e / dv, c = e - t * dv;
    vs[e] = A.v[(size_t)(t0 + t) * A.ldv + (size_t)h * dv + c];
  }
  __syncthreads();
  for (int c0 = 0; c0 < dv; c0 += VT) {
    const int c = c0 + 4 * lane;
    float4 s[ROWS > 0 ? ROWS : 1];
    if (ROWS > 0) {
#pragma unroll
      for (int i = 0; i < ROWS; ++i) {
        const int d = warp + 8 * i;
        s[i] = d < dk && c < dv ? la_load4(S + (size_t)d * dv, c, dv, vec) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
    for (int t = 0; t < n; ++t) {
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
      float4 vv;
      vv.x = c < dv ? vs[t * dv + c] : 0.f;
      vv.y = c + 1 < dv ? vs[t * dv + c + 1] : 0.f;
      vv.z = c + 2 < dv ? vs[t * dv + c + 2] : 0.f;
      vv.w = c + 3 < dv ? vs[t * dv + c + 3] : 0.f;
      auto step = [&](float4& x, int d) {
        const float kd = ks[t * dk + d], ed = es[t * dk + d], qd = qs[t * dk + d];
        x.x += fmaf(kd, vv.x, ed * x.x); x.y += fmaf(kd, vv.y, ed * x.y);
        x.z += fmaf(kd, vv.z, ed * x.z); x.w += fmaf(kd, vv.w, ed * x.w);
        o.x = fmaf(qd, x.x, o.x); o.y = fmaf(qd, x.y, o.y); o.z = fmaf(qd, x.z, o.z); o.w = fmaf(qd, x.w, o.w);
      };
      if (ROWS > 0) {
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
          const int d = warp + 8 * i;
          if (d < dk) step(s[i], d);
        }
      } else if (c < dv) {
        for (int d = warp; d < dk; d += 8) {
          float4 x = la_load4(S + (size_t)d * dv, c, dv, vec);
          step(x, d);
          la_store4(S + (size_t)d * dv, c, dv, vec, x);
        }
      }
      *reinterpret_cast<float4*>(part + warp * VT + 4 * lane) = o;
      __syncthreads();
      for (int e = threadIdx.x; e < VT && c0 + e < dv; e += blockDim.x) {
        float x = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) x += part[w * VT + e];
        os[t * dv + c0 + e] = x;
      }
      __syncthreads();
    }
    if (ROWS > 0) {
#pragma unroll
      for (int i = 0; i < ROWS; ++i) {
        const int d = warp + 8 * i;
        if (d < dk && c < dv) la_store4(S + (size_t)d * dv, c, dv, vec, s[i]);
      }
    }
  }
  for (int t = warp; t < n; t += 8) {
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) ss = fmaf(os[t * dv + c], os[t * dv + c], ss);
    ss = co_warp_sum(ss);
    const float sc = 1.0f / sqrtf(ss / (float)dv + A.eps);
    for (int c = lane; c < dv; c += 32) {
      const float gate = la_gate(A.gate_act, A.g[(size_t)(t0 + t) * A.ldg + (size_t)h * dv + c]);
      gla_store(A, t0 + t, (size_t)h * dv + c, ((os[t * dv + c] * sc) * co_load_any(A.norm_w, A.norm_dtype, c)) * gate);
    }
  }
}

// ------------------------------------------------------------------------------------------- chunks
// grid (ceil(T / 16), ceil(H dk / 128)), 128 threads: a thread takes one channel of sixteen tokens.
__global__ void __launch_bounds__(128) gla_decay_kernel(GlaArgs A) {
  extern __shared__ __align__(16) float sm[];      // [16][rank]
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int t0 = blockIdx.x * 16, n = min(16, A.T - t0);
  for (int e = threadIdx.x; e < 16 * A.rank; e += blockDim.x) {
    const int t = e / A.rank, r = e - t * A.rank;
    sm[e] = t < n ? A.a1[(size_t)(t0 + t) * A.lda + r] : 0.f;
  }
  __syncthreads();
  const size_t HK = (size_t)A.H * A.dk, ch = (size_t)blockIdx.y * 128 + threadIdx.x;
  if (ch >= HK) return;
  const float bias = A.a2b ? co_load_any(A.a2b, A.b_dtype, ch) : 0.f;
  float z[16];
#pragma unroll
  for (int t = 0; t < 16; ++t) z[t] = bias;
#pragma unroll 4
  for (int r = 0; r < A.rank; ++r) {
    const float w = co_load_any(A.a2, A.a2_dtype, ch * A.rank + r);
#pragma unroll
    for (int t = 0; t < 16; ++t) z[t] = fmaf(w, sm[t * A.rank + r], z[t]);
  }
#pragma unroll
  for (int t = 0; t < 16; ++t)
    if (t < n) A.log_decay[(size_t)(t0 + t) * HK + ch] = gla_log_decay(z[t], A.inv_tau);
}

struct Chunk {
  int first, n;       // first token of the step, tokens
  size_t index;       // row of the chunk areas
};
__device__ __forceinline__ Chunk gla_chunk(const GlaArgs& A, int r, int c) {
  const int q0 = A.cu_q[r], len = A.cu_q[r + 1] - q0;
  return {q0 + c * CH, min(CH, len - c * CH), (size_t)(q0 / CH + r + c)};
}

// grid (chunks of the longest run, B, H * ceil(dk / 64) * ceil(dv / VT)), 256 threads: a tile of 64 x 128 of the chunk's sum.
__global__ void __launch_bounds__(256) gla_chunk_state_kernel(GlaArgs A, bool vec) {
  extern __shared__ __align__(16) float sm[];
  float* Ks = sm;                    // [CH][68]
  float* Vs = Ks + CH * TP;          // [CH][VT]
  float* Ls = Vs + CH * VT;          // [64 channels][SP]: log decays, then the factors of the keys
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.y;
  const Chunk ck = gla_chunk(A, r, blockIdx.x);
  if (ck.n <= 0) return;
  const int dk = A.dk, dv = A.dv;
  const int nk = (dk + 63) / 64, nv = (dv + VT - 1) / VT;
  const int h = blockIdx.z / (nk * nv), kt = (blockIdx.z / nv) % nk, vt = blockIdx.z % nv;
  const int d0 = kt * 64, c0 = vt * VT;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll 8
  for (int i = 0; i < CH * 64 / 256; ++i) {
    const int e = threadIdx.x + 256 * i, t = e >> 6, d = e & 63;
    const bool in = t < ck.n && d0 + d < dk;
    const size_t ch = (size_t)h * dk + d0 + d, row = (size_t)ck.first + t;
    Ks[t * TP + d] = in ? A.k[row * A.ldk + ch] : 0.f;
    Ls[d * SP + t] = in ? A.log_decay[row * ((size_t)A.H * dk) + ch] : 0.f;
  }
#pragma unroll
  for (int i = 0; i < CH * (VT / 4) / 256; ++i) {
    const int e = threadIdx.x + 256 * i, t = e / (VT / 4), c4 = e % (VT / 4);
    const float4 x = t < ck.n ? la_load4(A.v + ((size_t)ck.first + t) * A.ldv + (size_t)h * dv, c0 + 4 * c4, dv, vec)
                              : make_float4(0.f, 0.f, 0.f, 0.f);
    *reinterpret_cast<float4*>(Vs + t * VT + 4 * c4) = x;
  }
  __syncthreads();
#pragma unroll 4
  for (int i = 0; i < 8; ++i) {          // a warp takes eight channels: sums of l over the tokens behind each token
    const int d = warp * 8 + i;
    float lo = Ls[d * SP + lane], hi = Ls[d * SP + 32 + lane];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float a = __shfl_down_sync(0xffffffffu, lo, o), c = __shfl_down_sync(0xffffffffu, hi, o);
      if (lane + o < 32) { lo += a; hi += c; }
    }
    const float total_hi = __shfl_sync(0xffffffffu, hi, 0), total = __shfl_sync(0xffffffffu, lo, 0) + total_hi;
    float xlo = __shfl_down_sync(0xffffffffu, lo, 1), xhi = __shfl_down_sync(0xffffffffu, hi, 1);
    if (lane == 31) { xlo = 0.f; xhi = 0.f; }
    Ls[d * SP + lane] = expf(xlo + total_hi);
    Ls[d * SP + 32 + lane] = expf(xhi);
    if (lane == 0 && vt == 0 && d0 + d < dk) A.chunk_decay[(ck.index * A.H + h) * dk + d0 + d] = total;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < CH * 64; e += 256) {
    const int t = e >> 6, d = e & 63;
    Ks[t * TP + d] *= Ls[d * SP + t];
  }
  __syncthreads();
  float acc[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  if (d0 + warp * 8 < dk) {
#pragma unroll 4
    for (int s = 0; s < ck.n; ++s) {
      const float4 k0 = *reinterpret_cast<const float4*>(Ks + s * TP + warp * 8);
      const float4 k1 = *reinterpret_cast<const float4*>(Ks + s * TP + warp * 8 + 4);
      const float4 x = *reinterpret_cast<const float4*>(Vs + s * VT + 4 * lane);
      const float kk[8] = {k0.x, k0.y, k0.z, k0.w, k1.x, k1.y, k1.z, k1.w};
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        acc[i][0] = fmaf(kk[i], x.x, acc[i][0]); acc[i][1] = fmaf(kk[i], x.y, acc[i][1]);
        acc[i][2] = fmaf(kk[i], x.z, acc[i][2]); acc[i][3] = fmaf(kk[i], x.w, acc[i][3]);
      }
    }
  }
  float* dst = A.chunk_state + (ck.index * A.H + h) * (size_t)dk * dv;
  const bool vs = (dv & 3) == 0;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int d = d0 + warp * 8 + i;
    if (d < dk && c0 + 4 * lane < dv)
      la_store4(dst + (size_t)d * dv, c0 + 4 * lane, dv, vs, make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]));
  }
}

// grid (ceil(dk * dv / (256 * W)), H, B), 256 threads, W elements each (4 when dv is a multiple of 4, else 1).
template <int W>
__global__ void __launch_bounds__(256) gla_state_scan_kernel(GlaArgs A) {
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.z, h = blockIdx.y;
  const int q0 = A.cu_q[r], len = A.cu_q[r + 1] - q0;
  if (len <= 0) return;
  const size_t size = (size_t)A.dk * A.dv;
  const size_t e = ((size_t)blockIdx.x * 256 + threadIdx.x) * W;
  if (e >= size) return;
  const int d = (int)(e / A.dv), chunks = (len + CH - 1) / CH;
  const size_t base = (size_t)(q0 / CH + r) * A.H + h;
  float* S = A.state + (size_t)A.state_slots[r] * A.state_stride + (size_t)h * size + e;
  float* cs = A.chunk_state + base * size + e;
  const float* cd = A.chunk_decay + base * A.dk + d;
  const size_t step = (size_t)A.H * size, dstep = (size_t)A.H * A.dk;
  float s[W];
#pragma unroll
  for (int i = 0; i < W; ++i) s[i] = S[i];
  constexpr int AHEAD = 4;
  for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
    float x[AHEAD][W], f[AHEAD];
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      if (c0 + a < chunks) {
        if (W == 4) *reinterpret_cast<float4*>(x[a]) = *reinterpret_cast<const float4*>(cs + (c0 + a) * step);
        else x[a][0] = cs[(c0 + a) * step];
        f[a] = cd[(c0 + a) * dstep];
      }
    }
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      if (c0 + a < chunks) {
        if (W == 4) *reinterpret_cast<float4*>(cs + (c0 + a) * step) = *reinterpret_cast<float4*>(s);
        else cs[(c0 + a) * step] = s[0];
        const float g = expm1f(f[a]);
#pragma unroll
        for (int i = 0; i < W; ++i) s[i] += fmaf(g, s[i], x[a][i]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < W; ++i) S[i] = s[i];
}

// grid (chunks of the longest run, B, H), 256 threads.
__global__ void __launch_bounds__(256, 2) gla_chunk_out_kernel(GlaArgs A, bool vec) {
  extern __shared__ __align__(16) float sm[];
  const int dk = A.dk, dv = A.dv;
  const int n_slices = (dk + SL - 1) / SL;
  float* QeT = sm;                               // [n_slices * SL][TP]: q exp(P)
  float* KeT = QeT + (size_t)n_slices * SL * TP; // [SL][TP]: k exp(-P)
  float* AsT = KeT + SL * TP;                    // [key][TP]: scores of a key for the chunk's tokens
  float* buf = AsT + CH * TP;                    // q, k, l slices [SL][SP] each; later two tiles [SL][VT]
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.y, h = blockIdx.z;
  const Chunk ck = gla_chunk(A, r, blockIdx.x);
  if (ck.n <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float* Qs = buf;
  float* Kst = Qs + SL * SP;
  float* Ls = Kst + SL * SP;
  for (int e = tid; e < CH * TP; e += 256) AsT[e] = 0.f;

  // scores: thread (ya, xa) of a 16 x 16 grid owns tokens 4 ya .. and keys 4 xa ..
  const int ya = tid >> 4, xa = tid & 15;
  float a[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) a[i][0] = a[i][1] = a[i][2] = a[i][3] = 0.f;
  float nq[CH / 8], nk[CH / 8], nl[CH / 8];      // the next slice's q, k, l: requested while the current one is used
  auto fetch_slice = [&](int sl) {
    const bool in_d = sl * SL + lane < dk;
    const size_t ch = (size_t)h * dk + sl * SL + lane;
#pragma unroll
    for (int i = 0; i < CH / 8; ++i) {
      const bool in = in_d && warp + 8 * i < ck.n;
      const size_t row = (size_t)ck.first + warp + 8 * i;
      nq[i] = in ? A.q[row * A.ldq + ch] : 0.f;
      nk[i] = in ? A.k[row * A.ldk + ch] : 0.f;
      nl[i] = in ? A.log_decay[row * ((size_t)A.H * dk) + ch] : 0.f;
    }
  };
  fetch_slice(0);
  for (int sl = 0; sl < n_slices; ++sl) {
    const int d0 = sl * SL;
#pragma unroll
    for (int i = 0; i < CH / 8; ++i) {
      const int t = warp + 8 * i;
      Qs[lane * SP + t] = nq[i] * A.q_scale;
      Kst[lane * SP + t] = nk[i];
      Ls[lane * SP + t] = nl[i];
    }
    __syncthreads();
    if (sl + 1 < n_slices) fetch_slice(sl + 1);
    bool far = false;
#pragma unroll
    for (int i = 0; i < SL / 8; ++i) {
      const int d = warp * (SL / 8) + i;
      float lo = Ls[d * SP + lane], hi = Ls[d * SP + 32 + lane];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, lo, o), y = __shfl_up_sync(0xffffffffu, hi, o);
        if (lane >= o) { lo += x; hi += y; }
      }
      hi += __shfl_sync(0xffffffffu, lo, 31);
      far |= __shfl_sync(0xffffffffu, hi, 31) < -FACTOR_LIMIT;
      QeT[(size_t)(d0 + d) * TP + lane] = Qs[d * SP + lane] * expf(lo);
      QeT[(size_t)(d0 + d) * TP + 32 + lane] = Qs[d * SP + 32 + lane] * expf(hi);
      KeT[d * TP + lane] = Kst[d * SP + lane] * expf(-lo);
      KeT[d * TP + 32 + lane] = Kst[d * SP + 32 + lane] * expf(-hi);
    }
    if (!__syncthreads_or(far)) {
      if (xa <= ya) {
#pragma unroll 8
        for (int d = 0; d < SL; ++d) {
          const float4 x = *reinterpret_cast<const float4*>(QeT + (size_t)(d0 + d) * TP + 4 * ya);
          const float4 y = *reinterpret_cast<const float4*>(KeT + d * TP + 4 * xa);
          const float xx[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            a[i][0] = fmaf(xx[i], y.x, a[i][0]); a[i][1] = fmaf(xx[i], y.y, a[i][1]);
            a[i][2] = fmaf(xx[i], y.z, a[i][2]); a[i][3] = fmaf(xx[i], y.w, a[i][3]);
          }
        }
      }
    } else {
      // a channel decays too far for the two factors: key s is carried forward by the tokens' own decays
      for (int e = tid; e < SL * CH; e += 256) Ls[(e / CH) * SP + e % CH] = expf(Ls[(e / CH) * SP + e % CH]);
      __syncthreads();
      const int s = tid >> 2, g = tid & 3;
      float ke[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) ke[j] = 0.f;
      for (int t = 0; t < CH; ++t) {
        float x = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const int d = g * 8 + j;
          ke[j] = t == s ? Kst[d * SP + s] : ke[j] * Ls[d * SP + t];
          x = fmaf(Qs[d * SP + t], ke[j], x);
        }
        x += __shfl_xor_sync(0xffffffffu, x, 1);
        x += __shfl_xor_sync(0xffffffffu, x, 2);
        if (g == 0 && t >= s) AsT[s * TP + t] += x;
      }
    }
    __syncthreads();
  }
  if (xa <= ya) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int s = 4 * xa + j;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = 4 * ya + i;
        if (s <= t) AsT[s * TP + t] += a[i][j];
      }
    }
  }

  // outputs: warp y owns tokens 8 y .., a lane four columns.  Left operands q exp(P) against the state the chunk starts
  // from (slices of SL key channels), then the scores against the values (two slices of SL tokens); the rows of the next
  // slice are fetched while the current one is used.
  const float* S0 = A.chunk_state + ((size_t)ck.index * A.H + h) * (size_t)dk * dv;
  const float* V0 = A.v + (size_t)ck.first * A.ldv + (size_t)h * dv;
  const bool vec_s = (dv & 3) == 0;
  const int total = n_slices + CH / SL;
  const size_t orow = (size_t)ck.first + warp * 8;
  float row_ss[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) row_ss[i] = 0.f;
  for (int c0 = 0; c0 < dv; c0 += VT) {
    float4 next[SL / 8];
    auto fetch = [&](int i) {
#pragma unroll
      for (int j = 0; j < SL / 8; ++j) {
        const int row = warp + 8 * j, c = c0 + 4 * lane;
        next[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < n_slices) {
          if (i * SL + row < dk && c < dv) next[j] = la_load4(S0 + (size_t)(i * SL + row) * dv, c, dv, vec_s);
        } else {
          const int t = (i - n_slices) * SL + row;
          if (t < ck.n && c < dv) next[j] = la_load4(V0 + (size_t)t * A.ldv, c, dv, vec);
        }
      }
    };
    auto put = [&](int i) {
      float* dst = buf + (i & 1) * SL * VT;
#pragma unroll
      for (int j = 0; j < SL / 8; ++j) *reinterpret_cast<float4*>(dst + (warp + 8 * j) * VT + 4 * lane) = next[j];
    };
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    fetch(0);
    __syncthreads();          // the scores are in place; nobody reads the tiles any more
    put(0);
    for (int i = 0; i < total; ++i) {
      __syncthreads();
      if (i + 1 < total) fetch(i + 1);
      const float* right = buf + (i & 1) * SL * VT + 4 * lane;
      const float* left = (i < n_slices ? QeT + (size_t)i * SL * TP : AsT + (i - n_slices) * SL * TP) + warp * 8;
      // a token's scores end at the token itself
      const int end = i < n_slices ? SL : min(SL, warp * 8 + 8 - (i - n_slices) * SL);
#pragma unroll 4
      for (int j = 0; j < end; ++j) {
        const float4 l0 = *reinterpret_cast<const float4*>(left + j * TP), l1 = *reinterpret_cast<const float4*>(left + j * TP + 4);
        const float4 x = *reinterpret_cast<const float4*>(right + j * VT);
        const float ll[8] = {l0.x, l0.y, l0.z, l0.w, l1.x, l1.y, l1.z, l1.w};
#pragma unroll
        for (int m = 0; m < 8; ++m) {
          acc[m][0] = fmaf(ll[m], x.x, acc[m][0]); acc[m][1] = fmaf(ll[m], x.y, acc[m][1]);
          acc[m][2] = fmaf(ll[m], x.z, acc[m][2]); acc[m][3] = fmaf(ll[m], x.w, acc[m][3]);
        }
      }
      if (i + 1 < total) put(i + 1);      // the other tile: its readers passed the barrier above
    }
    const int c = c0 + 4 * lane;
#pragma unroll
    for (int m = 0; m < 8; ++m)
      row_ss[m] += acc[m][0] * acc[m][0] + acc[m][1] * acc[m][1] + acc[m][2] * acc[m][2] + acc[m][3] * acc[m][3];
    if (dv > VT) {            // the rows' sums of squares are known behind the last tile only
#pragma unroll
      for (int m = 0; m < 8; ++m)
        if (warp * 8 + m < ck.n && c < dv)
          la_store4(A.o_raw + (orow + m) * ((size_t)A.H * dv) + (size_t)h * dv, c, dv, vec_s,
                     make_float4(acc[m][0], acc[m][1], acc[m][2], acc[m][3]));
      continue;
    }
#pragma unroll
    for (int m = 0; m < 8; ++m) {
      const float sc = 1.0f / sqrtf(co_warp_sum(row_ss[m]) / (float)dv + A.eps);
      if (warp * 8 + m >= ck.n) continue;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (c + e >= dv) break;
        const float gate = la_gate(A.gate_act, A.g[(orow + m) * A.ldg + (size_t)h * dv + c + e]);
        gla_store(A, orow + m, (size_t)h * dv + c + e, ((acc[m][e] * sc) * co_load_any(A.norm_w, A.norm_dtype, c + e)) * gate);
      }
    }
  }
  if (dv <= VT) return;
#pragma unroll
  for (int m = 0; m < 8; ++m) {
    const float sc = 1.0f / sqrtf(co_warp_sum(row_ss[m]) / (float)dv + A.eps);
    if (warp * 8 + m >= ck.n) continue;
    for (int c0 = 4 * lane; c0 < dv; c0 += VT) {          // what this thread wrote itself
      for (int e = 0; e < 4 && c0 + e < dv; ++e) {
        const int c = c0 + e;
        const float o = A.o_raw[(orow + m) * ((size_t)A.H * dv) + (size_t)h * dv + c];
        const float gate = la_gate(A.gate_act, A.g[(orow + m) * A.ldg + (size_t)h * dv + c]);
        gla_store(A, orow + m, (size_t)h * dv + c, ((o * sc) * co_load_any(A.norm_w, A.norm_dtype, c)) * gate);
      }
    }
  }
}

size_t few_smem(int L, int dk, int dv) { return ((size_t)8 * VT + (size_t)L * (3 * dk + 2 * dv)) * sizeof(float); }
size_t state_smem() { return ((size_t)CH * TP + (size_t)CH * VT + (size_t)64 * SP) * sizeof(float); }
size_t out_smem(int dk) {
  const size_t slices = (dk + SL - 1) / SL;
  const size_t tiles = 2 * SL * VT > 3 * SL * SP ? 2 * SL * VT : 3 * SL * SP;
  return (slices * SL * TP + (size_t)SL * TP + (size_t)CH * TP + tiles) * sizeof(float);
}
constexpr size_t SMEM_LIMIT = 220 * 1024;

}  // namespace

// Floats of scratch that a step needs (0: the kernel for few tokens per request, which needs none).
CO_EXPORT long coheryn_gla_scratch(int T, int B, int max_q_len, int few, int H, int dk, int dv) {
  if (max_q_len <= few) return 0;
  const long chunks = T / CH + B;
  return (long)T * H * dk + chunks * H * ((long)dk * dv + dk) + (dv > VT ? (long)T * H * dv : 0) + 8;
}

// few: requests of at most this many tokens take the kernel for few tokens (when the longest run of the step does).
CO_EXPORT int coheryn_gla(const float* q, long ldq, const float* k, long ldk, const float* v, long ldv, const float* g, long ldg,
                          const float* a1, long lda, const void* a2, int a2_dtype, const void* a2b, int b_dtype, int rank,
                          float tau, float q_scale, float* state, long state_stride, const int* cu_q, const int* state_slots,
                          const void* norm_w, int norm_dtype, float eps, int gate_act, void* out, int out_dtype, long ldo,
                          float* scratch, long scratch_floats, int T, int B, int H, int dk, int dv, int max_q_len, int few,
                          cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (dk < 1 || dv < 1 || H < 1 || rank < 1 || !(tau > 0.f)) CO_FAIL("gla: %d heads of %d x %d, rank %d, tau %g", H, dk, dv, rank, tau);
  if (out_dtype != CO_F32 && out_dtype != CO_BF16) CO_FAIL("gla: unknown output dtype %d", out_dtype);
  GlaArgs A{q, ldq, k, ldk, v, ldv, g, ldg, a1, lda, a2, a2_dtype, a2b, b_dtype, rank, 1.0f / tau, q_scale, state, state_stride, cu_q,
            state_slots, norm_w, norm_dtype, eps, gate_act, out, out_dtype, ldo, nullptr, nullptr, nullptr, nullptr, T, B, H, dk, dv};
  const auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  if (max_q_len <= few) {
    const size_t smem = few_smem(max_q_len, dk, dv);
    if (smem > SMEM_LIMIT) CO_FAIL("gla: %d tokens of heads %d x %d do not fit a CTA", max_q_len, dk, dv);
    const bool vec = (dv & 3) == 0 && (state_stride & 3) == 0 && aligned(state);
#define GO(ROWS)                                                                                                        \
  do {                                                                                                                  \
    if (smem > 48 * 1024) cudaFuncSetAttribute(gla_few_kernel<ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    co_launch(gla_few_kernel<ROWS>, dim3(H, B), dim3(256), smem, stream, A, max_q_len, vec);                            \
  } while (0)
    if (dk <= 32) GO(4); else if (dk <= 64) GO(8); else if (dk <= 128) GO(16); else if (dk <= 256) GO(32); else GO(0);
#undef GO
    CO_CHECK_LAUNCH("gla_few");
    return 0;
  }
  if (!scratch || scratch_floats < coheryn_gla_scratch(T, B, max_q_len, few, H, dk, dv)) CO_FAIL("gla: the scratch area is too small");
  if (out_smem(dk) > SMEM_LIMIT) CO_FAIL("gla: key heads of %d channels are not built for prompt portions", dk);
  const long chunks = T / CH + B;
  // the parts in order of their alignment needs: chunk states first
  A.chunk_state = scratch;
  A.o_raw = A.chunk_state + chunks * H * (long)dk * dv;
  A.chunk_decay = A.o_raw + (dv > VT ? (long)T * H * dv : 0);
  A.log_decay = A.chunk_decay + chunks * H * (long)dk;
  const bool vec = (ldv & 3) == 0 && (dv & 3) == 0 && aligned(v);
  const int per = (max_q_len + CH - 1) / CH, HK = H * dk;
  {
    const size_t smem = (size_t)16 * rank * sizeof(float);
    if (smem > SMEM_LIMIT) CO_FAIL("gla: a decay of rank %d is not built", rank);
    if (smem > 48 * 1024) cudaFuncSetAttribute(gla_decay_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    co_launch(gla_decay_kernel, dim3((T + 15) / 16, (HK + 127) / 128), dim3(128), smem, stream, A);
    CO_CHECK_LAUNCH("gla_decay");
  }
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(gla_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)state_smem());
    cudaFuncSetAttribute(gla_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM_LIMIT);
    configured = true;
  }
  co_launch(gla_chunk_state_kernel, dim3(per, B, H * ((dk + 63) / 64) * ((dv + VT - 1) / VT)), dim3(256), state_smem(), stream, A, vec);
  CO_CHECK_LAUNCH("gla_chunk_state");
  const size_t size = (size_t)dk * dv;
  if ((dv & 3) == 0 && (state_stride & 3) == 0 && aligned(state))
    co_launch(gla_state_scan_kernel<4>, dim3((unsigned)((size + 1023) / 1024), H, B), dim3(256), 0, stream, A);
  else
    co_launch(gla_state_scan_kernel<1>, dim3((unsigned)((size + 255) / 256), H, B), dim3(256), 0, stream, A);
  CO_CHECK_LAUNCH("gla_state_scan");
  co_launch(gla_chunk_out_kernel, dim3(per, B, H), dim3(256), out_smem(dk), stream, A, vec);
  CO_CHECK_LAUNCH("gla_chunk_out");
  return 0;
}
