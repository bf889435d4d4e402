// Generalised delta rule (fp32 state and recurrence; bf16 or fp32 projections).  Per head, with
//   u = k / sqrt(k.k + 1e-6),  w = exp(-e^(-1/2) sigmoid(w0 + low-rank projection)),  a = sigmoid(a + bias):
//   S <- diag(w) S - (a u)(u^T S) + k v^T,   o = S^T r.
// The columns of S (value channels) never meet, and the output needs no second pass over the new state:
//   o = (w r)^T S_old - (r . a u)(u^T S_old) + (r . k) v
// so one sweep over S yields both dot products and a second one updates it.
//   hy_delta_tanh    tanh of the low-rank decay projection, in place, ahead of its second matrix
//   hy_delta_scan    prompt portions, four tokens at a time; the state in registers, its columns spread over warps
//                    and blocks, while other warps prepare the next tokens (bf16, heads up to 128)
//   hy_delta_scan_any  the same with the state in shared memory: fp32, and other head sizes
//   hy_delta_decode  one token per sequence: the state is read and written once, norm and gate included
//   hy_delta_post    per head root-mean-square norm, gain, sigmoid gate -> the output projection's input
// In fp32 the decay is applied as S + (w - 1) S: where w is close to one its rounding to 32 bits would change
// the rate of a slow decay by 2^-25 / (1 - w).
// State: [slot][head][key][value] fp32; a sequence at position 0 starts from zeros whatever its slot holds.
#include "../common/host.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr float kDeltaUnit = 1e-6f;
constexpr float kDecayScale = 0.60653065971263342f;   // e^(-1/2)

template <typename T>
__global__ void __launch_bounds__(128)
hy_delta_tanh_kernel(T* __restrict__ proj, int ld, int off, int n, int rows) {
  const long t = (long)blockIdx.x * 128 + threadIdx.x;
  const int r = (int)(t / (n / 8)), i = (int)(t % (n / 8)) * 8;
  if (r >= rows) return;
  float f[8];
  load8(proj + (size_t)r * ld + off + i, f);
#pragma unroll
  for (int j = 0; j < 8; ++j) f[j] = tanhf(f[j]);
  store8(proj + (size_t)r * ld + off + i, f);
}

// What a token brings to one head, in shared memory: unit key, decay * r, decay (fp32: less one), k,
// removal (a u), v.
struct DeltaVecs {
  float *u, *wr, *w, *k, *au, *v;
  __device__ static DeltaVecs at(float* p, int n) { return {p, p + n, p + 2 * n, p + 3 * n, p + 4 * n, p + 5 * n}; }
};

// One warp turns the projections of a token into these vectors (zeros from D to DP); returns (r . a u, r . k)
// in every lane.
template <typename T>
__device__ __forceinline__ float2 delta_token(const BbHyLayer& L, const T* row, const T* low, int h, const DeltaVecs& s, int DP) {
  const int lane = threadIdx.x & 31, D = L.p, o = h * L.pp;
  float kk = 0.f;
  for (int d = lane; d < D; d += 32) {
    const float k = to_f(row[L.off_kk + o + d]);
    kk = fmaf(k, k, kk);
  }
  const float unit = 1.f / sqrtf(warp_sum(kk) + kDeltaUnit);
  float rau = 0.f, rk = 0.f;
  for (int d = lane; d < DP; d += 32) {
    const bool in = d < D;
    const float k = in ? to_f(row[L.off_kk + o + d]) : 0.f, r = in ? to_f(row[L.off_r + o + d]) : 0.f, u = k * unit;
    const float x = in ? -kDecayScale * sigmoid_as<T>(to_f(low[o + d]) + L.w0[o + d]) : 0.f;
    const float au = in ? sigmoid_as<T>(to_f(row[L.off_a + o + d]) + L.a_b[o + d]) * u : 0.f;
    const float w = sizeof(T) == 2 ? exp_hw(x) : expf(x);
    s.u[d] = u;
    s.wr[d] = w * r;
    s.w[d] = sizeof(T) == 2 ? w : expm1f(x);
    s.k[d] = k;
    s.au[d] = au;
    s.v[d] = in ? to_f(row[L.off_vv + o + d]) : 0.f;
    rau = fmaf(r, au, rau);
    rk = fmaf(r, k, rk);
  }
  return make_float2(warp_sum(rau), warp_sum(rk));
}
// New value of a state element.
template <typename T>
__device__ __forceinline__ float delta_apply(float w, float s, float k, float v, float au, float us) {
  const float t = fmaf(k, v, -au * us);
  return sizeof(T) == 2 ? fmaf(w, s, t) : s + fmaf(w, s, t);
}

// Any head size up to the shared memory: one block per (sequence, head), the state in shared memory, thread
// rows over keys and lanes over values.
constexpr int DS_THREADS = 256;

template <typename T>
__global__ void __launch_bounds__(DS_THREADS)
hy_delta_scan_any_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ low,
                         int ldl, T* __restrict__ y, int ldy, const __grid_constant__ BbHyBatch b, int seq0) {
  extern __shared__ __align__(16) float sm[];
  const int seq = seq0 + blockIdx.x, h = blockIdx.y, D = L.p;
  float* S = sm;                         // [D][D]
  float* vec = S + D * D;
  const DeltaVecs s = DeltaVecs::at(vec, D);
  __shared__ float dots[2];
  float* red = vec + 6 * D;              // [rows][2][D]
  int lanes = 1;
  while (lanes < D && lanes < 32) lanes <<= 1;
  const int lane = threadIdx.x % lanes, kr = threadIdx.x / lanes, rows = DS_THREADS / lanes;
  const int r0 = b.seq_row0[seq], r1 = b.seq_row0[seq + 1];
  float* state = L.ssm_state + ((size_t)b.seq_slot[seq] * L.heads + h) * D * D;
  const bool fresh = b.seq_pos0[seq] == 0;
  for (int i = threadIdx.x; i < D * D; i += DS_THREADS) S[i] = fresh ? 0.f : state[i];
  for (int r = r0; r < r1; ++r) {
    __syncthreads();
    if (threadIdx.x < 32) {
      const float2 d = delta_token<T>(L, proj + (size_t)r * ld, low + (size_t)r * ldl, h, s, D);
      if (threadIdx.x == 0) {
        dots[0] = d.x;
        dots[1] = d.y;
      }
    }
    __syncthreads();
    for (int j = lane; j < D; j += lanes) {
      float pu = 0.f, pr = 0.f;
      for (int i = kr; i < D; i += rows) {
        const float x = S[i * D + j];
        pu = fmaf(s.u[i], x, pu);
        pr = fmaf(s.wr[i], x, pr);
      }
      red[(kr * 2) * D + j] = pu;
      red[(kr * 2 + 1) * D + j] = pr;
    }
    __syncthreads();
    for (int j = lane; j < D; j += lanes) {
      float us = 0.f, os = 0.f;
      for (int q = 0; q < rows; ++q) {
        us += red[(q * 2) * D + j];
        os += red[(q * 2 + 1) * D + j];
      }
      const float v = s.v[j];
      if (kr == 0) y[(size_t)r * ldy + h * L.pp + j] = from_f<T>(fmaf(dots[1], v, fmaf(-dots[0], us, os)));
      for (int i = kr; i < D; i += rows) S[i * D + j] = delta_apply<T>(s.w[i], S[i * D + j], s.k[i], v, s.au[i], us);
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < D * D; i += DS_THREADS) state[i] = S[i];
}

// ---- state in registers, four tokens at a time.  With W_i..j the product of the decays of tokens i .. j of a
// group and S the state before it, the four dot products with the removed directions all run over the same S:
//   x_i = (W_0..i-1 u_i)^T S - sum_{j<i} (u_i . W_j+1..i-1 a_j u_j) x_j + sum_{j<i} (u_i . W_j+1..i-1 k_j) v_j
//   o_i = (W_0..i r_i)^T S   - sum_{j<=i} (r_i . W_j+1..i a_j u_j) x_j  + sum_{j<=i} (r_i . W_j+1..i k_j) v_j
//   S   <- W_0..3 S + sum_j (W_j+1..3 k_j) v_j^T - (W_j+1..3 a_j u_j) x_j^T
// (no decay is ever divided by).  The bracketed numbers do not depend on S: the warps that prepare a group have
// them ready, and one round of shuffles serves four tokens.  A thread holds four columns of eight keys, KL = DP / 8
// lanes a column: what bounds the kernel is the vectors' way from shared memory into registers, and every one of
// them then serves four columns.  Sums over keys end with a column to a lane, which solves for x and writes o.
constexpr int DG = 4;                                // tokens of a group

template <int DP>
struct DeltaGroup {
  // per group: U_i, R_i (4 each), W, K_j, A_j (4 each), v_j (4), then the 4 x 4 numbers of x (removal, value)
  // and of o
  static constexpr int U = 0, R = DG * DP, W = 2 * DG * DP, K = W + DP, A = K + DG * DP, V = A + DG * DP, X = V + DG * DP;
  static constexpr int SIZE = X + 64;
};

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("{\n\t.reg .b64 x, y, z;\n\t"
      "mov.b64 x, {%2, %3};\n\tmov.b64 y, {%4, %5};\n\tmov.b64 z, {%6, %7};\n\t"
      "fma.rn.f32x2 z, x, y, z;\n\t"
      "mov.b64 {%0, %1}, z;\n\t}"
      : "=f"(d.x), "=f"(d.y)
      : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
  return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
  float2 d;
  asm("{\n\t.reg .b64 x, y;\n\t"
      "mov.b64 x, {%2, %3};\n\tmov.b64 y, {%4, %5};\n\t"
      "mul.rn.f32x2 x, x, y;\n\t"
      "mov.b64 {%0, %1}, x;\n\t}"
      : "=f"(d.x), "=f"(d.y)
      : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
  return d;
}

// A group by one warp, DP / 32 neighbouring channels to a lane.
template <typename T, int DP>
struct DeltaPrep {
  using G = DeltaGroup<DP>;
  static constexpr int V = DP / 32;
  struct alignas(sizeof(T) * V) Raw {
    T v[V];
  };
  struct alignas(4 * V) Out {
    float v[V];
  };
  const BbHyLayer& L;
  const T *proj, *low;
  int ld, ldl, h;
  Raw r[DG], k[DG], v[DG], a[DG], x[DG];

  __device__ __forceinline__ void fetch(int r0, int t0, int n) {
    const int d = (threadIdx.x & 31) * V, o = h * L.pp + d;
    const bool in = d < L.pp;                        // (pp is a multiple of V)
    const T *row = proj + (size_t)(r0 + t0) * ld + o, *lrow = low + (size_t)(r0 + t0) * ldl + o;
#pragma unroll
    for (int i = 0; i < DG; ++i, row += ld, lrow += ldl) {
      if (in && t0 + i < n) {
        k[i] = *reinterpret_cast<const Raw*>(row + L.off_kk);
        r[i] = *reinterpret_cast<const Raw*>(row + L.off_r);
        v[i] = *reinterpret_cast<const Raw*>(row + L.off_vv);
        a[i] = *reinterpret_cast<const Raw*>(row + L.off_a);
        x[i] = *reinterpret_cast<const Raw*>(lrow);
        if (L.p != L.pp)
#pragma unroll
          for (int j = 0; j < V; ++j)
            if (d + j >= L.p) k[i].v[j] = r[i].v[j] = v[i].v[j] = from_f<T>(0.f);
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) k[i].v[j] = r[i].v[j] = v[i].v[j] = a[i].v[j] = x[i].v[j] = from_f<T>(0.f);
      }
    }
  }
  // Tokens past n leave the state as it is: their keys and values are zero and their decay is one.
  __device__ __forceinline__ void finish(float* p, int t0, int n) {
    if (t0 >= n) return;
    const int lane = threadIdx.x & 31, d = lane * V, o = h * L.pp + d;
    float s[32];
#pragma unroll
    for (int i = 0; i < DG; ++i) {
      s[i] = 0.f;
#pragma unroll
      for (int j = 0; j < V; ++j) s[i] = fmaf(to_f(k[i].v[j]), to_f(k[i].v[j]), s[i]);
    }
#pragma unroll
    for (int q = 16; q > 0; q >>= 1)
#pragma unroll
      for (int i = 0; i < DG; ++i) s[i] += __shfl_xor_sync(0xffffffffu, s[i], q);
    float unit[DG];
#pragma unroll
    for (int i = 0; i < DG; ++i) unit[i] = rsqrt_hw(s[i] + kDeltaUnit);
#pragma unroll
    for (int i = 0; i < 32; ++i) s[i] = 0.f;
    Out O[3 * DG + 1 + 2 * DG];                      // U, R, W, K, A in the group's order, then v
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float w0 = d < L.pp ? L.w0[o + j] : 0.f, ab = d < L.pp ? L.a_b[o + j] : 0.f;
      float w[DG], u[DG], rr[DG], kk[DG], au[DG];
#pragma unroll
      for (int i = 0; i < DG; ++i) {
        w[i] = t0 + i < n ? exp2_hw(-kDecayScale * kLog2e * sigmoid_as<T>(to_f(x[i].v[j]) + w0)) : 1.f;
        kk[i] = to_f(k[i].v[j]);
        rr[i] = to_f(r[i].v[j]);
        u[i] = kk[i] * unit[i];
        au[i] = sigmoid_as<T>(to_f(a[i].v[j]) + ab) * u[i];
      }
      // numbers: row i of x at 0 (removal) and 6 (value), of o at 12 and 22
      int nx = 0, no = 0;
      float before = 1.f;
#pragma unroll
      for (int i = 0; i < DG; ++i) {
        O[i].v[j] = before * u[i];
        before *= w[i];
        O[DG + i].v[j] = before * rr[i];
      }
      O[2 * DG].v[j] = before;
#pragma unroll
      for (int i = 0; i < DG; ++i) {
        float au_w[DG], k_w[DG];                     // vectors of earlier tokens as token i finds them
#pragma unroll
        for (int q = 0; q < DG; ++q) {
          if (q >= i) continue;
          float m = 1.f;
#pragma unroll
          for (int e = 0; e < DG; ++e)
            if (e > q && e < i) m *= w[e];
          au_w[q] = m * au[q];
          k_w[q] = m * kk[q];
          s[nx] = fmaf(u[i], au_w[q], s[nx]);
          s[6 + nx] = fmaf(u[i], k_w[q], s[6 + nx]);
          ++nx;
        }
#pragma unroll
        for (int q = 0; q < DG; ++q) {
          if (q > i) continue;
          const float rw = q < i ? rr[i] * w[i] : rr[i];
          s[12 + no] = fmaf(rw, q < i ? au_w[q] : au[q], s[12 + no]);
          s[22 + no] = fmaf(rw, q < i ? k_w[q] : kk[q], s[22 + no]);
          ++no;
        }
      }
#pragma unroll
      for (int q = 0; q < DG; ++q) {
        float m = 1.f;
#pragma unroll
        for (int e = 0; e < DG; ++e)
          if (e > q) m *= w[e];
        O[2 * DG + 1 + q].v[j] = m * kk[q];
        O[3 * DG + 1 + q].v[j] = m * au[q];
        O[4 * DG + 1 + q].v[j] = to_f(v[q].v[j]);
      }
    }
#pragma unroll
    for (int i = 0; i < 5 * DG + 1; ++i) *reinterpret_cast<Out*>(p + i * DP + d) = O[i];
    // 32 sums over the warp, sum i to lane i
#pragma unroll
    for (int c = 16; c > 0; c >>= 1) {
      const bool up = lane & c;
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        if (i >= c) break;
        const float keep = up ? s[i + c] : s[i], send = up ? s[i] : s[i + c];
        s[i] = keep + __shfl_xor_sync(0xffffffffu, send, c);
      }
    }
    // ... and into the 4 x 4 tables (their other places stay zero)
    const int set = lane < 6 ? 0 : (lane < 12 ? 1 : (lane < 22 ? 2 : 3));
    const int e = lane - (set == 0 ? 0 : (set == 1 ? 6 : (set == 2 ? 12 : 22)));
    int i, q;
    if (set < 2) {
      i = e == 0 ? 1 : (e < 3 ? 2 : 3);
      q = e - i * (i - 1) / 2;
    } else {
      i = e == 0 ? 0 : (e < 3 ? 1 : (e < 6 ? 2 : 3));
      q = e - i * (i + 1) / 2;
    }
    p[G::X + set * 16 + i * 4 + q] = s[0];
  }
};

// CW warps walk through the tokens, PREP others prepare one group each of the buffer that comes next; BLOCKS of
// them are to share an SM.
template <typename T, int DP, int CW, int PREP, int BLOCKS>
__global__ void __launch_bounds__((CW + PREP) * 32, BLOCKS)
hy_delta_scan_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ low,
                     int ldl, T* __restrict__ y, int ldy, const __grid_constant__ BbHyBatch b) {
  using G = DeltaGroup<DP>;
  constexpr int KL = DP / 8, CT = 4, STEP = DG * PREP, NT = DG * 4 / KL;   // NT: tokens whose outputs a lane finishes
  static_assert(KL >= 4 && NT >= 1, "a lane for every column of a thread");
  constexpr int COLS = CW * (32 / KL) * CT;          // columns of a block
  extern __shared__ __align__(16) float sm[];        // [2][PREP][G::SIZE]
  const int seq = blockIdx.z, h = blockIdx.y, D = L.p;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r0 = b.seq_row0[seq], n = b.seq_row0[seq + 1] - r0;
  for (int i = threadIdx.x; i < 2 * PREP * 64; i += blockDim.x) sm[(i / 64) * G::SIZE + G::X + i % 64] = 0.f;
  __syncthreads();
  if (warp >= CW) {
    DeltaPrep<T, DP> prep{L, proj, low, ld, ldl, h};
    const int w = warp - CW;
    prep.fetch(r0, w * DG, n);
    prep.finish(sm + w * G::SIZE, w * DG, n);
    prep.fetch(r0, STEP + w * DG, n);
    __syncthreads();
    for (int t0 = 0, it = 1; t0 < n; t0 += STEP, ++it) {
      const int t = t0 + STEP + w * DG;
      prep.finish(sm + ((it & 1) * PREP + w) * G::SIZE, t, n);
      prep.fetch(r0, t + STEP, n);
      __syncthreads();
    }
    return;
  }
  // keys 4 q .. 4 q + 3 and DP / 2 + 4 q .. of columns c0 .. c0 + 3
  const int q = lane % KL, c0 = blockIdx.x * COLS + (warp * (32 / KL) + lane / KL) * CT;
  float* state = L.ssm_state + ((size_t)b.seq_slot[seq] * L.heads + h) * D * D;
  const bool fresh = b.seq_pos0[seq] == 0;
  float2 S[CT][4];                                   // two neighbouring keys of a column
  auto key = [&](int i) { return (i / 2) * (DP / 2) + 4 * q + 2 * (i & 1); };
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int c = 0; c < CT; ++c) {
      const int k = key(i), col = c0 + c;
      S[c][i].x = !fresh && k < D && col < D ? state[(size_t)k * D + col] : 0.f;
      S[c][i].y = !fresh && k + 1 < D && col < D ? state[(size_t)(k + 1) * D + col] : 0.f;
    }
  const int cv = min(c0, DP - CT), col = q & 3, tok = (q >> 2) * NT;   // this lane's column and first output token
  const bool b1 = q & 2, b0 = q & 1;
  T* yt = y + (size_t)(r0 + tok) * ldy + h * L.pp + c0 + col;   // first output of this lane in the group at hand
  const bool writes = c0 < L.pp;                     // (pp is a multiple of 4: all four columns or none)
  __syncthreads();
  for (int t0 = 0, it = 0; t0 < n; t0 += STEP, ++it) {
    const float* p = sm + (it & 1) * PREP * G::SIZE;
    for (int t = t0; t < min(t0 + STEP, n); t += DG, p += G::SIZE) {
      auto vec = [&](int off, int m) { return reinterpret_cast<const float4*>(p + off + m * (DP / 2))[q]; };
      auto dots = [&](int off, float (&out)[CT]) {
        float2 acc[CT];
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          const float4 u = vec(off, m);
#pragma unroll
          for (int c = 0; c < CT; ++c) {
            acc[c] = m ? fma2(make_float2(u.x, u.y), S[c][2], acc[c]) : mul2(make_float2(u.x, u.y), S[c][0]);
            acc[c] = fma2(make_float2(u.z, u.w), S[c][2 * m + 1], acc[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < CT; ++c) out[c] = acc[c].x + acc[c].y;
      };
      // in phases, so that the latency of one token's shuffles and loads covers the others'
      float x[DG], o[DG], v[DG];                     // of this lane's column
      float f[DG][CT], g[DG][CT];
#pragma unroll
      for (int i = 0; i < DG; ++i) dots(G::U + i * DP, f[i]);
#pragma unroll
      for (int i = 0; i < DG; ++i) {
        f[i][0] = (b1 ? f[i][2] : f[i][0]) + __shfl_xor_sync(0xffffffffu, b1 ? f[i][0] : f[i][2], 2);
        f[i][1] = (b1 ? f[i][3] : f[i][1]) + __shfl_xor_sync(0xffffffffu, b1 ? f[i][1] : f[i][3], 2);
      }
#pragma unroll
      for (int i = 0; i < DG; ++i) dots(G::R + i * DP, g[i]);
#pragma unroll
      for (int i = 0; i < DG; ++i) x[i] = (b0 ? f[i][1] : f[i][0]) + __shfl_xor_sync(0xffffffffu, b0 ? f[i][0] : f[i][1], 1);
#pragma unroll
      for (int i = 0; i < DG; ++i) v[i] = p[G::V + i * DP + cv + col];
      float ca[DG][DG], cw[DG][DG];
#pragma unroll
      for (int i = 1; i < DG; ++i) {
        const float4 ra = *reinterpret_cast<const float4*>(p + G::X + i * 4), rv = *reinterpret_cast<const float4*>(p + G::X + 16 + i * 4);
        ca[i][0] = ra.x; ca[i][1] = ra.y; ca[i][2] = ra.z; ca[i][3] = ra.w;
        cw[i][0] = rv.x; cw[i][1] = rv.y; cw[i][2] = rv.z; cw[i][3] = rv.w;
      }
#pragma unroll
      for (int d = 4; d < KL; d <<= 1)
#pragma unroll
        for (int i = 0; i < DG; ++i) x[i] += __shfl_xor_sync(0xffffffffu, x[i], d);
#pragma unroll
      for (int i = 0; i < DG; ++i) {
        g[i][0] = (b1 ? g[i][2] : g[i][0]) + __shfl_xor_sync(0xffffffffu, b1 ? g[i][0] : g[i][2], 2);
        g[i][1] = (b1 ? g[i][3] : g[i][1]) + __shfl_xor_sync(0xffffffffu, b1 ? g[i][1] : g[i][3], 2);
      }
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const float4 w = vec(G::W, m);
#pragma unroll
        for (int c = 0; c < CT; ++c) {
          S[c][2 * m] = mul2(make_float2(w.x, w.y), S[c][2 * m]);
          S[c][2 * m + 1] = mul2(make_float2(w.z, w.w), S[c][2 * m + 1]);
        }
      }
#pragma unroll
      for (int i = 0; i < DG; ++i) o[i] = (b0 ? g[i][1] : g[i][0]) + __shfl_xor_sync(0xffffffffu, b0 ? g[i][0] : g[i][1], 1);
      // ... NT tokens to a lane
#pragma unroll
      for (int d = KL / 2, c = DG / 2; d >= 4; d >>= 1, c >>= 1) {
        const bool up = q & d;
#pragma unroll
        for (int i = 0; i < DG / 2; ++i)
          if (i < c) {
            const float keep = up ? o[i + c] : o[i], send = up ? o[i] : o[i + c];
            o[i] = keep + __shfl_xor_sync(0xffffffffu, send, d);
          }
      }
      float4 ga[NT];
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        ga[i] = *reinterpret_cast<const float4*>(p + G::X + 32 + (tok + i) * 4);
        const float4 gv = *reinterpret_cast<const float4*>(p + G::X + 48 + (tok + i) * 4);
        o[i] = (o[i] + fmaf(gv.y, v[1], gv.x * v[0])) + fmaf(gv.w, v[3], gv.z * v[2]);
      }
      // the part of the update and of x that the values alone make
#pragma unroll
      for (int j = 0; j < DG; ++j) {
        const float4 v4 = *reinterpret_cast<const float4*>(p + G::V + j * DP + cv);
        const float vc[CT] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          const float4 k = vec(G::K + j * DP, m);
#pragma unroll
          for (int c = 0; c < CT; ++c) {
            const float2 vv = make_float2(vc[c], vc[c]);
            S[c][2 * m] = fma2(make_float2(k.x, k.y), vv, S[c][2 * m]);
            S[c][2 * m + 1] = fma2(make_float2(k.z, k.w), vv, S[c][2 * m + 1]);
          }
        }
      }
#pragma unroll
      for (int i = 1; i < DG; ++i)
#pragma unroll
        for (int j = 0; j < i; ++j) x[i] = fmaf(cw[i][j], v[j], x[i]);
#pragma unroll
      for (int i = 1; i < DG; ++i)
#pragma unroll
        for (int j = 0; j < i; ++j) x[i] = fmaf(-ca[i][j], x[j], x[i]);
      // every lane gets the x of its four columns, and the state moves on
      float lo[DG], hi[DG], xc[DG][CT];
#pragma unroll
      for (int j = 0; j < DG; ++j) {
        const float n1 = __shfl_xor_sync(0xffffffffu, x[j], 1);
        lo[j] = b0 ? n1 : x[j];
        hi[j] = b0 ? x[j] : n1;
      }
#pragma unroll
      for (int j = 0; j < DG; ++j) {
        const float lo2 = __shfl_xor_sync(0xffffffffu, lo[j], 2), hi2 = __shfl_xor_sync(0xffffffffu, hi[j], 2);
        xc[j][0] = b1 ? lo2 : lo[j];
        xc[j][1] = b1 ? hi2 : hi[j];
        xc[j][2] = b1 ? lo[j] : lo2;
        xc[j][3] = b1 ? hi[j] : hi2;
      }
      // outputs, while the shuffles are on their way
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const float f = fmaf(-ga[i].y, x[1], fmaf(-ga[i].x, x[0], o[i])) - fmaf(ga[i].w, x[3], ga[i].z * x[2]);
        if (writes && t + tok + i < n) yt[i * ldy] = from_f<T>(f);
      }
      yt += DG * (size_t)ldy;
#pragma unroll
      for (int j = 0; j < DG; ++j)
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          const float4 a = vec(G::A + j * DP, m);
#pragma unroll
          for (int c = 0; c < CT; ++c) {
            const float2 xx = make_float2(-xc[j][c], -xc[j][c]);
            S[c][2 * m] = fma2(make_float2(a.x, a.y), xx, S[c][2 * m]);
            S[c][2 * m + 1] = fma2(make_float2(a.z, a.w), xx, S[c][2 * m + 1]);
          }
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int c = 0; c < CT; ++c) {
      const int k = key(i), cl = c0 + c;
      if (k < D && cl < D) state[(size_t)k * D + cl] = S[c][i].x;
      if (k + 1 < D && cl < D) state[(size_t)(k + 1) * D + cl] = S[c][i].y;
    }
}

// ---- one token per sequence.  Lanes over four columns each, thread rows over keys, U keys of a thread.
template <typename T, int THREADS, int U>
__global__ void __launch_bounds__(THREADS)
hy_delta_decode_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ low,
                       int ldl, T* __restrict__ cat, int ldc, const __grid_constant__ BbHyBatch b, float eps) {
  extern __shared__ __align__(16) float sm[];
  const int seq = b.ns_pre + blockIdx.x, h = blockIdx.y, D = L.p, cv = D / 4;
  const size_t r = b.n_pre + blockIdx.x;
  int lanes = 1;
  while (lanes < cv) lanes <<= 1;
  const int lane = threadIdx.x % lanes, kr = threadIdx.x / lanes, rows = THREADS / lanes;
  const DeltaVecs s = DeltaVecs::at(sm, D);
  float* red = sm + 6 * D;                           // [rows][2][D]
  float* out = red + rows * 2 * D;                   // [D]
  __shared__ float dots[2];
  float* state = L.ssm_state + ((size_t)b.seq_slot[seq] * L.heads + h) * D * D;
  const bool fresh = b.pos[r] == 0, mine = lane < cv;
  float4 S[U];
#pragma unroll
  for (int i = 0; i < U; ++i) {
    const int k = kr + i * rows;
    S[i] = !fresh && mine && k < D ? reinterpret_cast<const float4*>(state + (size_t)k * D)[lane] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (threadIdx.x < 32) {
    const float2 d = delta_token<T>(L, proj + r * ld, low + r * ldl, h, s, D);
    if (threadIdx.x == 0) {
      dots[0] = d.x;
      dots[1] = d.y;
    }
  }
  __syncthreads();
  float4 pu = make_float4(0.f, 0.f, 0.f, 0.f), pr = pu;
#pragma unroll
  for (int i = 0; i < U; ++i) {
    const int k = kr + i * rows;
    if (k < D) {
      const float u = s.u[k], w = s.wr[k];
      pu.x = fmaf(u, S[i].x, pu.x); pu.y = fmaf(u, S[i].y, pu.y); pu.z = fmaf(u, S[i].z, pu.z); pu.w = fmaf(u, S[i].w, pu.w);
      pr.x = fmaf(w, S[i].x, pr.x); pr.y = fmaf(w, S[i].y, pr.y); pr.z = fmaf(w, S[i].z, pr.z); pr.w = fmaf(w, S[i].w, pr.w);
    }
  }
  if (mine) {
    reinterpret_cast<float4*>(red + (kr * 2) * D)[lane] = pu;
    reinterpret_cast<float4*>(red + (kr * 2 + 1) * D)[lane] = pr;
  }
  __syncthreads();
  if (mine) {
    float4 us = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int q = 0; q < rows; ++q) {
      const float4 a = reinterpret_cast<const float4*>(red + (q * 2) * D)[lane];
      us.x += a.x; us.y += a.y; us.z += a.z; us.w += a.w;
    }
    const float4 v = reinterpret_cast<const float4*>(s.v)[lane];
    if (kr == 0) {
      float4 os = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int q = 0; q < rows; ++q) {
        const float4 a = reinterpret_cast<const float4*>(red + (q * 2 + 1) * D)[lane];
        os.x += a.x; os.y += a.y; os.z += a.z; os.w += a.w;
      }
      // the same rounding of the recurrence's output as in a prompt portion
      auto fin = [&](float o, float u, float x) { return to_f(from_f<T>(fmaf(dots[1], x, fmaf(-dots[0], u, o)))); };
      reinterpret_cast<float4*>(out)[lane] =
          make_float4(fin(os.x, us.x, v.x), fin(os.y, us.y, v.y), fin(os.z, us.z, v.z), fin(os.w, us.w, v.w));
    }
#pragma unroll
    for (int i = 0; i < U; ++i) {
      const int k = kr + i * rows;
      if (k < D) {
        const float w = s.w[k], kk = s.k[k], au = s.au[k];
        reinterpret_cast<float4*>(state + (size_t)k * D)[lane] =
            make_float4(delta_apply<T>(w, S[i].x, kk, v.x, au, us.x), delta_apply<T>(w, S[i].y, kk, v.y, au, us.y),
                        delta_apply<T>(w, S[i].z, kk, v.z, au, us.z), delta_apply<T>(w, S[i].w, kk, v.w, au, us.w));
      }
    }
  }
  __syncthreads();
  if (threadIdx.x < 32) {
    const int o = h * L.pp;
    float ss = 0.f;
    for (int d = threadIdx.x; d < D; d += 32) ss = fmaf(out[d], out[d], ss);
    const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)D + eps);
    for (int d = threadIdx.x; d < L.pp; d += 32)
      cat[r * ldc + o + d] = from_f<T>(
          d < D ? out[d] * rstd * L.gnorm[o + d] * sigmoid_as<T>(to_f(proj[r * ld + L.off_gg + o + d])) : 0.f);
  }
}

// One block per row; a head's vectors of 8 lie in `lanes` neighbouring threads (a power of two up to 32).
constexpr int DPOST_THREADS = 256;

template <typename T>
__global__ void __launch_bounds__(DPOST_THREADS)
hy_delta_post_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ y, int ldy,
                     T* __restrict__ cat, int ldc, int lanes, float eps) {
  const size_t r = blockIdx.x;
  const int lane = threadIdx.x % lanes, vecs = L.pp / 8;
  for (int h = threadIdx.x / lanes; h < ((L.heads + DPOST_THREADS / lanes - 1) & ~(DPOST_THREADS / lanes - 1));
       h += DPOST_THREADS / lanes) {
    const bool live = h < L.heads;
    float ss = 0.f, f[8], g[8], w[8];
    auto load = [&](int v) {
      const int o = h * L.pp + v * 8;
      load8(y + r * ldy + o, f);
      load8(proj + r * ld + L.off_gg + o, g);
      load8(L.gnorm + o, w);
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (v * 8 + j >= L.p) f[j] = 0.f;
    };
    for (int v = lane; live && v < vecs; v += lanes) {
      load(v);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
    }
    for (int o = 1; o < lanes; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float rstd = 1.f / sqrtf(ss / (float)L.p + eps);
    for (int v = lane; live && v < vecs; v += lanes) {
      if (vecs > lanes) load(v);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= rstd * w[j] * sigmoid_as<T>(g[j]);
      store8(cat + r * ldc + h * L.pp + v * 8, f);
    }
  }
}

template <typename T>
static int launch_scan_any(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, int seq0, int n_seq, cudaStream_t s) {
  static PerDeviceOnce once;
  int lanes = 1;
  while (lanes < L.p && lanes < 32) lanes <<= 1;
  const size_t smem = 4ull * ((size_t)L.p * L.p + 6 * L.p + 2 * (DS_THREADS / lanes) * (size_t)L.p);
  if (smem > 220 * 1024) return BB_ESIZE;
  const cudaError_t e = ensure_dyn_smem(once, hy_delta_scan_any_kernel<T>, 220 * 1024);
  if (e != cudaSuccess) return (int)e;
  hy_delta_scan_any_kernel<T><<<dim3(n_seq, L.heads), DS_THREADS, smem, s>>>(
      L, static_cast<const T*>(w.proj), w.ld_proj, static_cast<const T*>(w.aux), w.ld_aux, static_cast<T*>(w.y), w.ld_y, b, seq0);
  return (int)cudaGetLastError();
}

template <int DP, int CW, int PREP, int BLOCKS>
static int launch_scan_regs(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, cudaStream_t s) {
  using T = __nv_bfloat16;
  static PerDeviceOnce once;
  constexpr int smem = 2 * PREP * DeltaGroup<DP>::SIZE * 4, cols = CW * (32 / (DP / 8)) * 4;
  const cudaError_t e = ensure_dyn_smem(once, hy_delta_scan_kernel<T, DP, CW, PREP, BLOCKS>, smem);
  if (e != cudaSuccess) return (int)e;
  hy_delta_scan_kernel<T, DP, CW, PREP, BLOCKS><<<dim3((L.p + cols - 1) / cols, L.heads, b.ns_pre), (CW + PREP) * 32, smem, s>>>(
      L, static_cast<const T*>(w.proj), w.ld_proj, static_cast<const T*>(w.aux), w.ld_aux, static_cast<T*>(w.y), w.ld_y, b);
  return (int)cudaGetLastError();
}

// Few heads: the columns of a head are spread over more blocks.  Many: two blocks share an SM.
static int launch_scan_bf16(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, cudaStream_t s) {
  const long pairs = (long)b.ns_pre * L.heads;
  const int sms = sm_count();
  if (L.p <= 32) return launch_scan_regs<32, 1, 8, 2>(L, w, b, s);
  if (L.p <= 64) {
    if (pairs * 4 <= sms) return launch_scan_regs<64, 1, 8, 1>(L, w, b, s);
    if (pairs * 2 <= sms) return launch_scan_regs<64, 2, 8, 1>(L, w, b, s);
    return pairs <= sms ? launch_scan_regs<64, 4, 8, 1>(L, w, b, s) : launch_scan_regs<64, 4, 6, 2>(L, w, b, s);
  }
  if (L.p <= 128) return pairs * 8 <= sms ? launch_scan_regs<128, 2, 8, 1>(L, w, b, s) : launch_scan_regs<128, 4, 8, 1>(L, w, b, s);
  return BB_ESIZE;
}

template <typename T, int THREADS, int U>
static int launch_decode_u(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, float eps, cudaStream_t s) {
  int lanes = 1;
  while (lanes < L.p / 4) lanes <<= 1;
  const size_t smem = 4ull * (7 + 2 * (THREADS / lanes)) * L.p;
  if (smem > 48 * 1024) return BB_ESIZE;
  hy_delta_decode_kernel<T, THREADS, U><<<dim3(b.ns - b.ns_pre, L.heads), THREADS, smem, s>>>(
      L, static_cast<const T*>(w.proj), w.ld_proj, static_cast<const T*>(w.aux), w.ld_aux, static_cast<T*>(w.cat), w.ld_cat, b, eps);
  return (int)cudaGetLastError();
}
template <typename T>
static int launch_decode(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, float eps, cudaStream_t s) {
  if (L.p % 4 || L.p > 128) return BB_ESIZE;
  if (L.p <= 32) return launch_decode_u<T, 128, 2>(L, w, b, eps, s);
  if (L.p <= 64) return launch_decode_u<T, 128, 8>(L, w, b, eps, s);
  return launch_decode_u<T, 256, 16>(L, w, b, eps, s);
}

template <typename T>
static int launch_post(const BbHyLayer& L, const BbHyWork& w, int rows, float eps, cudaStream_t s) {
  int lanes = 1;
  while (lanes < L.pp / 8 && lanes < 32) lanes <<= 1;
  hy_delta_post_kernel<T><<<rows, DPOST_THREADS, 0, s>>>(L, static_cast<const T*>(w.proj), w.ld_proj,
                                                         static_cast<const T*>(w.y), w.ld_y, static_cast<T*>(w.cat), w.ld_cat,
                                                         lanes, eps);
  return (int)cudaGetLastError();
}

template <typename T>
static int run_delta(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, float eps, cudaStream_t s) {
  const int n_dec = b.ns - b.ns_pre;
  int post = b.n_pre;                    // rows whose outputs are still to be normed and gated
  if (n_dec > 0) {
    int rc = launch_decode<T>(L, w, b, eps, s);
    if (rc == BB_ESIZE) {
      rc = launch_scan_any<T>(L, w, b, b.ns_pre, n_dec, s);
      post = b.n;
    }
    if (rc) return rc;
  }
  if (b.ns_pre > 0) {
    int rc = sizeof(T) == 2 ? launch_scan_bf16(L, w, b, s) : BB_ESIZE;
    if (rc == BB_ESIZE) rc = launch_scan_any<T>(L, w, b, 0, b.ns_pre, s);
    if (rc) return rc;
  }
  return post > 0 ? launch_post<T>(L, w, post, eps, s) : BB_OK;
}

}  // namespace bb

using namespace bb;

BB_API int bb_hy_delta_tanh(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  const long t = (long)b->n * (L->wrp / 8);
  const int grid = (int)((t + 127) / 128);
  cudaStream_t s = (cudaStream_t)stream;
  if (c->dtype) hy_delta_tanh_kernel<float><<<grid, 128, 0, s>>>(static_cast<float*>(w->proj), w->ld_proj, L->off_w1, L->wrp, b->n);
  else hy_delta_tanh_kernel<__nv_bfloat16><<<grid, 128, 0, s>>>(static_cast<__nv_bfloat16*>(w->proj), w->ld_proj, L->off_w1, L->wrp, b->n);
  return (int)cudaGetLastError();
}

// Recurrence, norm and gate of every row of the step -> w->cat.
BB_API int bb_hy_delta(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  return c->dtype ? run_delta<float>(*L, *w, *b, c->eps, (cudaStream_t)stream)
                  : run_delta<__nv_bfloat16>(*L, *w, *b, c->eps, (cudaStream_t)stream);
}

// Norm and gate of the first `rows` rows of w->y -> w->cat: any recurrence whose heads end that way.
BB_API int bb_hy_head_post(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int rows, void* stream) {
  if (rows <= 0) return BB_OK;
  return c->dtype ? launch_post<float>(*L, *w, rows, c->eps, (cudaStream_t)stream)
                  : launch_post<__nv_bfloat16>(*L, *w, rows, c->eps, (cudaStream_t)stream);
}

// The recurrence of the prompt portions alone -> w->y; `any`: by the kernel that covers every size.
BB_API int bb_hy_delta_scan(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int any, void* stream) {
  cudaStream_t s = (cudaStream_t)stream;
  if (b->ns_pre <= 0) return BB_OK;
  if (c->dtype) return launch_scan_any<float>(*L, *w, *b, 0, b->ns_pre, s);
  return any ? launch_scan_any<__nv_bfloat16>(*L, *w, *b, 0, b->ns_pre, s) : launch_scan_bf16(*L, *w, *b, s);
}
