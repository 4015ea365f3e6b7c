// Linear attention with a constant decay per head (sm_100a, float32 throughout): per request and head a state S [dk, dv],
//
//   S_t = a S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,      q, k, v: the projections, each passed through SiLU (optional),
//   out_t = o_t / rms(o_t over ALL heads together) * w * act(g_t) * factor;      act = sigmoid or SiLU.
//
// Powers of the decays come from the host, made in float64: [head][2][CH + 1] floats, a^n and a^n - 1.
//
// Two ways to the same numbers, chosen by the longest run of tokens a request brings:
//
//   * lightning_few_kernel (decoding, portions of a few tokens): a CTA per (head, 32 value channels, request) holds its part
//     of S in registers and takes the tokens one by one.  S changes by (a - 1) S + k v^T, so that a decay near 1 keeps its
//     digits.
//   * chunks of 64 tokens (prompt portions), counted from a request's first token of the step:
//       lightning_chunk_state_kernel  per (chunk, head): sum_s a^(n-1-s) k_s v_s^T over the chunk's n tokens;
//       lightning_state_scan_kernel   over a request's chunks: the state every chunk starts from; the last one is stored;
//       lightning_chunk_out_kernel    per (chunk, head): o_t = a^(t+1) S_start^T q_t + sum_{s <= t} a^(t-s) (q_t . k_s) v_s.
//
// Both leave o in float32; lightning_norm_kernel (a CTA per token) sees all heads of a token and writes the output.
// A row's order of additions is fixed by its place in its request's run, not by what else the step holds.
#include "linear_attention.cuh"

namespace {

constexpr int CH = 64;            // tokens per chunk
constexpr int TP = CH + 4;        // pitch of a [channel][token] tile that is read four tokens at a time
constexpr int SL = 32;            // channels (or tokens) per slice of the output kernel
constexpr int FC = 32;            // value channels per CTA of the kernel for few tokens, times its column groups

struct LightningArgs {
  const float* q; long ldq; const float* k; long ldk; const float* v; long ldv;
  const float* powers;    // [H][2][CH + 1]
  int silu;               // whether q, k and v pass SiLU on their way in
  float* state; long state_stride;
  const int* cu_q; const int* state_slots;
  float* chunk_state;     // [T / CH + B][H][dk][dv]: request r's chunk c is row cu_q[r] / CH + r + c
  float* o_raw;           // [T][H dv]
  int T, B, H, dk, dv;
};

__device__ __forceinline__ float li_act(int silu, float z) { return silu ? __fdividef(z, 1.0f + expf(-z)) : z; }
__device__ __forceinline__ float4 li_act4(int silu, float4 z) {
  return make_float4(li_act(silu, z.x), li_act(silu, z.y), li_act(silu, z.z), li_act(silu, z.w));
}
__device__ __forceinline__ void li_axpy(float4& o, float a, const float4& x) {
  o.x = fmaf(a, x.x, o.x); o.y = fmaf(a, x.y, o.y); o.z = fmaf(a, x.z, o.z); o.w = fmaf(a, x.w, o.w);
}

// ------------------------------------------------------------------------------------------- few tokens per request
// grid (H, ceil(dv / (FC NC)), B), 256 threads.  Eight neighbouring lanes own four columns each of every column group; lane
// group g of the 32 owns the rows g, g + 32, .. of S.  ROWS: rows a thread keeps in registers (0: the state stays in memory,
// for dk > 256).  NC: column groups of a CTA (two where many heads and requests fill the GPU by themselves).
// smem: q, k [L][dk], v [L][CW], the warps' partial outputs [L][8][CW]; L = tokens of the longest run.
template <int ROWS, int NC>
__global__ void __launch_bounds__(256, NC == 2 ? 3 : 1) lightning_few_kernel(LightningArgs A, int L, bool vec) {
  constexpr int CW = FC * NC;
  extern __shared__ __align__(16) float sm[];
  co_pdl_launch_dependents();
  const int h = blockIdx.x, c0 = blockIdx.y * CW, b = blockIdx.z, dk = A.dk, dv = A.dv;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = threadIdx.x >> 3, c = c0 + 4 * (lane & 7);
  float* part = sm;                     // [L][8][CW]
  float* vs = part + L * 8 * CW;        // [L][CW]
  float* qs = vs + L * CW;
  float* ks = qs + L * dk;
  const float am1 = A.powers[(size_t)h * 2 * (CH + 1) + CH + 1 + 1];
  co_pdl_wait();
  const int t0 = A.cu_q[b], n = A.cu_q[b + 1] - t0;
  if (n <= 0) return;
  float* S = A.state + (size_t)A.state_slots[b] * A.state_stride + (size_t)h * dk * dv;
  float4 s[ROWS > 0 ? ROWS : 1][NC];
  if (ROWS > 0) {                       // in flight while the projections are read
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int d = g + 32 * i;
#pragma unroll
      for (int j = 0; j < NC; ++j)
        s[i][j] = d < dk && c + FC * j < dv ? la_load4(S + (size_t)d * dv, c + FC * j, dv, vec) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  for (int e = threadIdx.x; e < n * dk; e += 256) {
    const int t = e / dk, d = e - t * dk;
    const size_t row = t0 + t, ch = (size_t)h * dk + d;
    qs[e] = li_act(A.silu, A.q[row * A.ldq + ch]);
    ks[e] = li_act(A.silu, A.k[row * A.ldk + ch]);
  }
  for (int e = threadIdx.x; e < n * CW; e += 256) {
    const int t = e / CW, x = e - t * CW;
    vs[e] = c0 + x < dv ? li_act(A.silu, A.v[(size_t)(t0 + t) * A.ldv + (size_t)h * dv + c0 + x]) : 0.f;
  }
  __syncthreads();
  for (int t = 0; t < n; ++t) {
#pragma unroll
    for (int j = 0; j < NC; ++j) {
      const float4 vv = *reinterpret_cast<const float4*>(vs + t * CW + FC * j + 4 * (lane & 7));
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
      auto step = [&](float4& x, int d) {
        const float kd = ks[t * dk + d], qd = qs[t * dk + d];
        x.x += fmaf(kd, vv.x, am1 * x.x); x.y += fmaf(kd, vv.y, am1 * x.y);
        x.z += fmaf(kd, vv.z, am1 * x.z); x.w += fmaf(kd, vv.w, am1 * x.w);
        li_axpy(o, qd, x);
      };
      if (ROWS > 0) {
#pragma unroll
        for (int i = 0; i < ROWS; ++i)
          if (g + 32 * i < dk) step(s[i][j], g + 32 * i);
      } else if (c + FC * j < dv) {
        for (int d = g; d < dk; d += 32) {
          float4 x = la_load4(S + (size_t)d * dv, c + FC * j, dv, vec);
          step(x, d);
          la_store4(S + (size_t)d * dv, c + FC * j, dv, vec, x);
        }
      }
#pragma unroll
      for (int off = 8; off < 32; off <<= 1) {       // the warp's four lane groups
        o.x += __shfl_xor_sync(0xffffffffu, o.x, off); o.y += __shfl_xor_sync(0xffffffffu, o.y, off);
        o.z += __shfl_xor_sync(0xffffffffu, o.z, off); o.w += __shfl_xor_sync(0xffffffffu, o.w, off);
      }
      if (lane < 8) *reinterpret_cast<float4*>(part + (t * 8 + warp) * CW + FC * j + 4 * lane) = o;
    }
  }
  if (ROWS > 0) {
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int d = g + 32 * i;
#pragma unroll
      for (int j = 0; j < NC; ++j)
        if (d < dk && c + FC * j < dv) la_store4(S + (size_t)d * dv, c + FC * j, dv, vec, s[i][j]);
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < n * CW; e += 256) {
    const int t = e / CW, x = e - t * CW;
    if (c0 + x >= dv) continue;
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) o += part[(t * 8 + w) * CW + x];
    A.o_raw[(size_t)(t0 + t) * ((size_t)A.H * dv) + (size_t)h * dv + c0 + x] = o;
  }
}

// ------------------------------------------------------------------------------------------- chunks
struct Chunk {
  int first, n;       // first token of the step, tokens
  size_t index;       // row of the chunk area
};
__device__ __forceinline__ Chunk li_chunk(const LightningArgs& A, int r, int c) {
  const int q0 = A.cu_q[r], len = A.cu_q[r + 1] - q0;
  return {q0 + c * CH, min(CH, len - c * CH), (size_t)(q0 / CH + r + c)};
}

// CPL neighbouring columns per lane: a tile of 32 CPL value channels.
template <int CPL> struct Cols;
template <> struct Cols<4> {
  float4 x;
  __device__ __forceinline__ void zero() { x = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ void get(const float* p) { x = *reinterpret_cast<const float4*>(p); }
  __device__ __forceinline__ void axpy(float a, const Cols& y) { li_axpy(x, a, y.x); }
  __device__ __forceinline__ void times(float a) { x.x *= a; x.y *= a; x.z *= a; x.w *= a; }
  __device__ __forceinline__ float at(int i) const { return i == 0 ? x.x : i == 1 ? x.y : i == 2 ? x.z : x.w; }
};
template <> struct Cols<2> {
  float2 x;
  __device__ __forceinline__ void zero() { x = make_float2(0.f, 0.f); }
  __device__ __forceinline__ void get(const float* p) { x = *reinterpret_cast<const float2*>(p); }
  __device__ __forceinline__ void axpy(float a, const Cols& y) { x.x = fmaf(a, y.x.x, x.x); x.y = fmaf(a, y.x.y, x.y); }
  __device__ __forceinline__ void times(float a) { x.x *= a; x.y *= a; }
  __device__ __forceinline__ float at(int i) const { return i == 0 ? x.x : x.y; }
};
template <int CPL>
__device__ __forceinline__ void li_store(float* row, int c, int n, bool vec, const Cols<CPL>& y) {
  if constexpr (CPL == 4) {
    la_store4(row, c, n, vec, y.x);
  } else {
    if (vec && c + 1 < n) { *reinterpret_cast<float2*>(row + c) = y.x; return; }
    if (c < n) row[c] = y.x.x;
    if (c + 1 < n) row[c + 1] = y.x.y;
  }
}

// grid (chunks of the longest run, B, H * ceil(dk / 64) * ceil(dv / VT)), 256 threads: a tile of 64 x VT of the chunk's sum.
template <int CPL>
__global__ void __launch_bounds__(256) lightning_chunk_state_kernel(LightningArgs A, bool veck, bool vec) {
  constexpr int VT = 32 * CPL;
  extern __shared__ __align__(16) float sm[];
  float* Ks = sm;                    // [CH][64]: keys times the decay behind them
  float* Vs = Ks + CH * 64;          // [CH][VT]
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.y;
  const Chunk ck = li_chunk(A, r, blockIdx.x);
  if (ck.n <= 0) return;
  const int dk = A.dk, dv = A.dv;
  const int nk = (dk + 63) / 64, nv = (dv + VT - 1) / VT;
  const int h = blockIdx.z / (nk * nv), kt = (blockIdx.z / nv) % nk, vt = blockIdx.z % nv;
  const int d0 = kt * 64, c0 = vt * VT;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float* pw = A.powers + (size_t)h * 2 * (CH + 1);
#pragma unroll
  for (int i = 0; i < CH * 16 / 256; ++i) {
    const int e = threadIdx.x + 256 * i, t = e >> 4, d = 4 * (e & 15);
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (t < ck.n) {
      x = li_act4(A.silu, la_load4(A.k + ((size_t)ck.first + t) * A.ldk + (size_t)h * dk, d0 + d, dk, veck));
      const float f = pw[ck.n - 1 - t];
      x = make_float4(x.x * f, x.y * f, x.z * f, x.w * f);
    }
    *reinterpret_cast<float4*>(Ks + t * 64 + d) = x;
  }
#pragma unroll
  for (int i = 0; i < CH * (VT / 4) / 256; ++i) {
    const int e = threadIdx.x + 256 * i, t = e / (VT / 4), c4 = e % (VT / 4);
    *reinterpret_cast<float4*>(Vs + t * VT + 4 * c4) =
        t < ck.n ? li_act4(A.silu, la_load4(A.v + ((size_t)ck.first + t) * A.ldv + (size_t)h * dv, c0 + 4 * c4, dv, vec))
                 : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  __syncthreads();
  if (d0 + warp * 8 >= dk) return;
  Cols<CPL> acc[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i].zero();
#pragma unroll 4
  for (int s = 0; s < ck.n; ++s) {
    const float4 k0 = *reinterpret_cast<const float4*>(Ks + s * 64 + warp * 8);
    const float4 k1 = *reinterpret_cast<const float4*>(Ks + s * 64 + warp * 8 + 4);
    Cols<CPL> x;
    x.get(Vs + s * VT + CPL * lane);
    const float kk[8] = {k0.x, k0.y, k0.z, k0.w, k1.x, k1.y, k1.z, k1.w};
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i].axpy(kk[i], x);
  }
  float* dst = A.chunk_state + (ck.index * A.H + h) * (size_t)dk * dv;
  const bool vs = (dv & 3) == 0;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int d = d0 + warp * 8 + i;
    if (d < dk && c0 + CPL * lane < dv) li_store<CPL>(dst + (size_t)d * dv, c0 + CPL * lane, dv, vs, acc[i]);
  }
}

// grid (ceil(dk * dv / (256 * W)), H, B), 256 threads, W elements each (4 when the sizes allow it, else 1).
template <int W>
__global__ void __launch_bounds__(256) lightning_state_scan_kernel(LightningArgs A) {
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.z, h = blockIdx.y;
  const int q0 = A.cu_q[r], len = A.cu_q[r + 1] - q0;
  if (len <= 0) return;
  const size_t size = (size_t)A.dk * A.dv;
  const size_t e = ((size_t)blockIdx.x * 256 + threadIdx.x) * W;
  if (e >= size) return;
  const int chunks = (len + CH - 1) / CH;
  const float* m1 = A.powers + (size_t)h * 2 * (CH + 1) + CH + 1;
  const float whole = m1[CH], last = m1[len - (chunks - 1) * CH];
  float* S = A.state + (size_t)A.state_slots[r] * A.state_stride + (size_t)h * size + e;
  float* cs = A.chunk_state + ((size_t)(q0 / CH + r) * A.H + h) * size + e;
  const size_t step = (size_t)A.H * size;
  float s[W];
#pragma unroll
  for (int i = 0; i < W; ++i) s[i] = S[i];
  constexpr int AHEAD = 8;
  for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
    float x[AHEAD][W];
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      if (c0 + a < chunks) {
        if (W == 4) *reinterpret_cast<float4*>(x[a]) = *reinterpret_cast<const float4*>(cs + (c0 + a) * step);
        else x[a][0] = cs[(c0 + a) * step];
      }
    }
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      if (c0 + a < chunks) {
        if (W == 4) *reinterpret_cast<float4*>(cs + (c0 + a) * step) = *reinterpret_cast<float4*>(s);
        else cs[(c0 + a) * step] = s[0];
        const float f = c0 + a == chunks - 1 ? last : whole;
#pragma unroll
        for (int i = 0; i < W; ++i) s[i] += fmaf(f, s[i], x[a][i]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < W; ++i) S[i] = s[i];
}

// grid (chunks of the longest run, B, H), 256 threads.
template <int CPL>
__global__ void __launch_bounds__(256, 2) lightning_chunk_out_kernel(LightningArgs A, bool vec) {
  constexpr int VT = 32 * CPL;
  extern __shared__ __align__(16) float sm[];
  const int dk = A.dk, dv = A.dv;
  const int n_slices = (dk + SL - 1) / SL;
  float* QT = sm;                                // [n_slices * SL][TP]
  float* AsT = QT + (size_t)n_slices * SL * TP;  // [key][TP]: a^(t-s) (q_t . k_s) of a key for the chunk's tokens
  float* buf = AsT + CH * TP;                    // key slices [2][SL][TP]; later two tiles [SL][VT]
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.y, h = blockIdx.z;
  const Chunk ck = li_chunk(A, r, blockIdx.x);
  if (ck.n <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const float* pw = A.powers + (size_t)h * 2 * (CH + 1);

  // scores: thread (ya, xa) of a 16 x 16 grid owns tokens 4 ya .. and keys 4 xa ..
  const int ya = tid >> 4, xa = tid & 15;
  float a[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) a[i][0] = a[i][1] = a[i][2] = a[i][3] = 0.f;
  float nq[CH / 8], nk[CH / 8];      // the next slice's q, k: requested while the current one is used
  auto fetch_slice = [&](int sl) {
    const bool in_d = sl * SL + lane < dk;
    const size_t ch = (size_t)h * dk + sl * SL + lane;
#pragma unroll
    for (int i = 0; i < CH / 8; ++i) {
      const bool in = in_d && warp + 8 * i < ck.n;
      const size_t row = (size_t)ck.first + warp + 8 * i;
      nq[i] = in ? A.q[row * A.ldq + ch] : 0.f;
      nk[i] = in ? A.k[row * A.ldk + ch] : 0.f;
    }
  };
  fetch_slice(0);
  for (int sl = 0; sl < n_slices; ++sl) {
    float* Kt = buf + (sl & 1) * SL * TP;
#pragma unroll
    for (int i = 0; i < CH / 8; ++i) {
      const int t = warp + 8 * i;
      QT[(size_t)(sl * SL + lane) * TP + t] = li_act(A.silu, nq[i]);
      Kt[lane * TP + t] = li_act(A.silu, nk[i]);
    }
    __syncthreads();
    if (sl + 1 < n_slices) fetch_slice(sl + 1);
    if (xa <= ya) {
#pragma unroll 8
      for (int d = 0; d < SL; ++d) {
        const float4 x = *reinterpret_cast<const float4*>(QT + (size_t)(sl * SL + d) * TP + 4 * ya);
        const float4 y = *reinterpret_cast<const float4*>(Kt + d * TP + 4 * xa);
        const float xx[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          a[i][0] = fmaf(xx[i], y.x, a[i][0]); a[i][1] = fmaf(xx[i], y.y, a[i][1]);
          a[i][2] = fmaf(xx[i], y.z, a[i][2]); a[i][3] = fmaf(xx[i], y.w, a[i][3]);
        }
      }
    }
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int s = 4 * xa + j;
    float4 x;
    float* xp = &x.x;
#pragma unroll
    for (int i = 0; i < 4; ++i) xp[i] = s <= 4 * ya + i ? a[i][j] * pw[4 * ya + i - s] : 0.f;
    *reinterpret_cast<float4*>(AsT + s * TP + 4 * ya) = x;
  }

  // outputs: warp y owns tokens 8 y .., a lane CPL columns.  First q against the state the chunk starts from (slices of SL
  // key channels), times a^(t+1), then the scores against the values (two slices of SL tokens); the rows of the next slice
  // are fetched while the current one is used.
  const float* S0 = A.chunk_state + ((size_t)ck.index * A.H + h) * (size_t)dk * dv;
  const float* V0 = A.v + (size_t)ck.first * A.ldv + (size_t)h * dv;
  const bool vec_s = (dv & 3) == 0;
  const int total = n_slices + (ck.n + SL - 1) / SL;
  const size_t orow = (size_t)ck.first + warp * 8;
  constexpr int R4 = SL * (VT / 4) / 256;         // float4 a thread moves per slice
  for (int c0 = 0; c0 < dv; c0 += VT) {
    float4 next[R4];
    auto fetch = [&](int i) {
#pragma unroll
      for (int j = 0; j < R4; ++j) {
        const int e = tid + 256 * j, row = e / (VT / 4), c = c0 + 4 * (e % (VT / 4));
        next[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < n_slices) {
          if (i * SL + row < dk && c < dv) next[j] = la_load4(S0 + (size_t)(i * SL + row) * dv, c, dv, vec_s);
        } else {
          const int t = (i - n_slices) * SL + row;
          if (t < ck.n && c < dv) next[j] = li_act4(A.silu, la_load4(V0 + (size_t)t * A.ldv, c, dv, vec));
        }
      }
    };
    auto put = [&](int i) {
      float* dst = buf + (i & 1) * SL * VT;
#pragma unroll
      for (int j = 0; j < R4; ++j) *reinterpret_cast<float4*>(dst + 4 * (tid + 256 * j)) = next[j];
    };
    Cols<CPL> acc[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i].zero();
    fetch(0);
    __syncthreads();          // the scores are in place; nobody reads the tiles any more
    put(0);
    for (int i = 0; i < total; ++i) {
      __syncthreads();
      if (i + 1 < total) fetch(i + 1);
      if (i == n_slices) {
#pragma unroll
        for (int m = 0; m < 8; ++m) acc[m].times(pw[warp * 8 + m + 1]);
      }
      const float* right = buf + (i & 1) * SL * VT + CPL * lane;
      const float* left = (i < n_slices ? QT + (size_t)i * SL * TP : AsT + (i - n_slices) * SL * TP) + warp * 8;
      // a token's scores end at the token itself
      const int end = i < n_slices ? SL : min(SL, warp * 8 + 8 - (i - n_slices) * SL);
#pragma unroll 4
      for (int j = 0; j < end; ++j) {
        const float4 l0 = *reinterpret_cast<const float4*>(left + j * TP), l1 = *reinterpret_cast<const float4*>(left + j * TP + 4);
        Cols<CPL> x;
        x.get(right + j * VT);
        const float ll[8] = {l0.x, l0.y, l0.z, l0.w, l1.x, l1.y, l1.z, l1.w};
#pragma unroll
        for (int m = 0; m < 8; ++m) acc[m].axpy(ll[m], x);
      }
      if (i + 1 < total) put(i + 1);      // the other tile: its readers passed the barrier above
    }
    const int c = c0 + CPL * lane;
#pragma unroll
    for (int m = 0; m < 8; ++m)
      if (warp * 8 + m < ck.n && c < dv) li_store<CPL>(A.o_raw + (orow + m) * ((size_t)A.H * dv) + (size_t)h * dv, c, dv, vec_s, acc[m]);
  }
}

// grid (T), 256 threads: all heads of a token normalised together, times the weight, the gate and a factor.
template <typename TO>
__global__ void __launch_bounds__(256) lightning_norm_kernel(const float* __restrict__ o, const void* __restrict__ w, int w_dtype,
                                                             const float* __restrict__ gate, long ldg, int gate_act, float eps,
                                                             float factor, TO* __restrict__ out, long ldo, int n) {
  extern __shared__ __align__(16) float row_s[];      // [n]
  __shared__ float scratch[33];
  co_pdl_launch_dependents();
  co_pdl_wait();
  const size_t t = blockIdx.x;
  float ss = 0.f;
  for (int j = threadIdx.x; j < n; j += blockDim.x) {
    const float x = o[t * n + j];
    row_s[j] = x;
    ss = fmaf(x, x, ss);
  }
  const float inv = 1.0f / sqrtf(co_block_sum(ss, scratch) / (float)n + eps);
  for (int j = threadIdx.x; j < n; j += blockDim.x)
    out[t * ldo + j] = co_from_float<TO>((row_s[j] * inv) * co_load_any(w, w_dtype, j) * la_gate(gate_act, gate[t * ldg + j]) * factor);
}

size_t few_smem(int L, int dk, int columns) { return ((size_t)L * 9 * columns + (size_t)2 * L * dk) * sizeof(float); }
size_t state_smem(int vt) { return ((size_t)CH * 64 + (size_t)CH * vt) * sizeof(float); }
size_t out_smem(int dk, int vt) {
  const size_t slices = (dk + SL - 1) / SL, tiles = (size_t)2 * SL * vt, keys = (size_t)2 * SL * TP;
  return (slices * SL * TP + (size_t)CH * TP + (tiles > keys ? tiles : keys)) * sizeof(float);
}
constexpr size_t SMEM_LIMIT = 220 * 1024;

}  // namespace

// Tokens per chunk: the powers reach from 0 to it.
CO_EXPORT int coheryn_lightning_chunk() { return CH; }

// Floats of scratch that a step needs.
CO_EXPORT long coheryn_lightning_scratch(int T, int B, int max_q_len, int few, int H, int dk, int dv) {
  const long chunks = max_q_len <= few ? 0 : T / CH + B;
  return chunks * H * (long)dk * dv + (long)T * H * dv;
}

// few: requests of at most this many tokens take the kernel for few tokens (when the longest run of the step does).
CO_EXPORT int coheryn_lightning(const float* q, long ldq, const float* k, long ldk, const float* v, long ldv, const float* gate,
                                long ldg, const float* powers, int silu, float* state, long state_stride, const int* cu_q,
                                const int* state_slots, const void* norm_w, int norm_dtype, float eps, int gate_act, float factor,
                                void* out, int out_dtype, long ldo, float* scratch, long scratch_floats, int T, int B, int H, int dk,
                                int dv, int max_q_len, int few, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (dk < 1 || dv < 1 || H < 1) CO_FAIL("lightning: %d heads of %d x %d", H, dk, dv);
  if (out_dtype != CO_F32 && out_dtype != CO_BF16) CO_FAIL("lightning: unknown output dtype %d", out_dtype);
  if (!powers || !norm_w || !gate) CO_FAIL("lightning: powers, norm weight and gate are needed");
  if (!scratch || scratch_floats < coheryn_lightning_scratch(T, B, max_q_len, few, H, dk, dv)) CO_FAIL("lightning: the scratch area is too small");
  LightningArgs A{q, ldq, k, ldk, v, ldv, powers, silu, state, state_stride, cu_q, state_slots, nullptr, nullptr, T, B, H, dk, dv};
  const auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool vec_state = (dv & 3) == 0 && (state_stride & 3) == 0 && aligned(state);
  if (max_q_len <= few) {
    A.o_raw = scratch;
    // twice the columns per CTA once three rounds of the narrow ones would be needed
    const bool wide = dk <= 128 && dv > FC && (long)H * ((dv + FC - 1) / FC) * B > 3 * 148 * 2;
    const size_t smem = few_smem(max_q_len, dk, wide ? 2 * FC : FC);
    if (smem > SMEM_LIMIT) CO_FAIL("lightning: %d tokens of %d key channels do not fit a CTA", max_q_len, dk);
#define GO(ROWS, NC)                                                                                                          \
  do {                                                                                                                        \
    if (smem > 48 * 1024) cudaFuncSetAttribute(lightning_few_kernel<ROWS, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    co_launch(lightning_few_kernel<ROWS, NC>, dim3(H, (dv + FC * NC - 1) / (FC * NC), B), dim3(256), smem, stream, A, max_q_len, vec_state); \
  } while (0)
    if (wide) { if (dk <= 32) GO(1, 2); else if (dk <= 64) GO(2, 2); else GO(4, 2); }
    else if (dk <= 32) GO(1, 1); else if (dk <= 64) GO(2, 1); else if (dk <= 128) GO(4, 1); else if (dk <= 256) GO(8, 1); else GO(0, 1);
#undef GO
    CO_CHECK_LAUNCH("lightning_few");
  } else {
    const int vt = dv <= 64 ? 64 : 128;
    const size_t smem = out_smem(dk, vt);
    if (smem > SMEM_LIMIT) CO_FAIL("lightning: key heads of %d channels are not built for prompt portions", dk);
    const long chunks = T / CH + B;
    A.chunk_state = scratch;
    A.o_raw = scratch + chunks * H * (long)dk * dv;
    const bool veck = (ldk & 3) == 0 && (dk & 3) == 0 && aligned(k), vec = (ldv & 3) == 0 && (dv & 3) == 0 && aligned(v);
    const int per = (max_q_len + CH - 1) / CH;
    const size_t size = (size_t)dk * dv;
    const dim3 sgrid(per, B, H * ((dk + 63) / 64) * ((dv + vt - 1) / vt)), ogrid(per, B, H);
    cudaFuncSetAttribute(lightning_chunk_state_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)state_smem(128));
    if (vt == 64) co_launch(lightning_chunk_state_kernel<2>, sgrid, dim3(256), state_smem(64), stream, A, veck, vec);
    else co_launch(lightning_chunk_state_kernel<4>, sgrid, dim3(256), state_smem(128), stream, A, veck, vec);
    CO_CHECK_LAUNCH("lightning_chunk_state");
    if (vec_state && aligned(scratch)) co_launch(lightning_state_scan_kernel<4>, dim3((unsigned)((size + 1023) / 1024), H, B), dim3(256), 0, stream, A);
    else co_launch(lightning_state_scan_kernel<1>, dim3((unsigned)((size + 255) / 256), H, B), dim3(256), 0, stream, A);
    CO_CHECK_LAUNCH("lightning_state_scan");
    if (vt == 64) {
      cudaFuncSetAttribute(lightning_chunk_out_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM_LIMIT);
      co_launch(lightning_chunk_out_kernel<2>, ogrid, dim3(256), smem, stream, A, vec);
    } else {
      cudaFuncSetAttribute(lightning_chunk_out_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM_LIMIT);
      co_launch(lightning_chunk_out_kernel<4>, ogrid, dim3(256), smem, stream, A, vec);
    }
    CO_CHECK_LAUNCH("lightning_chunk_out");
  }
  const int n = H * dv;
  const size_t smem = (size_t)n * sizeof(float);
  if (smem > SMEM_LIMIT) CO_FAIL("lightning: %d value channels of all heads do not fit a CTA", n);
#define GO(TO)                                                                                                                \
  do {                                                                                                                        \
    if (smem > 48 * 1024) cudaFuncSetAttribute(lightning_norm_kernel<TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    co_launch(lightning_norm_kernel<TO>, dim3(T), dim3(256), smem, stream, (const float*)A.o_raw, norm_w, norm_dtype, gate, ldg, \
              gate_act, eps, factor, (TO*)out, ldo, n);                                                                       \
  } while (0)
  if (out_dtype == CO_F32) GO(float); else GO(__nv_bfloat16);
#undef GO
  CO_CHECK_LAUNCH("lightning_norm");
  return 0;
}
