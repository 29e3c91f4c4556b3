// Linear recurrences whose decay and input strength are numbers per (token, head), float32 throughout:
//
//     S <- exp(x_t) S + b_t k v^T,   o = S^T q                      S: [key dim x value dim] per head, x_t <= 0
//
// in two forms that differ in where x and b come from and in what is made of o:
//
//   state space (Mamba-2's scalar decay):  dt = softplus(raw + bias);  x = -exp(A_log) dt,  b = dt;
//                                          out = o + D v             (k, q are shared by the heads of a group)
//   matrix memory (mLSTM):  i = cap tanh((raw_i + bias_i) / cap),  f = logsigmoid(cap tanh((raw_f + bias_f) / cap)),
//                           m <- max(f + m, i),  x = f + m_old - m,  b = exp(i - m);  n <- exp(x) n + b k;
//                           out = o,  den = max(|n . q|, exp(-m)) + 1e-6      (who normalises the heads divides by den)
//
// A step holds portions of several requests (qo_indptr, state_slots).  Every sum runs in an order fixed by the sizes alone, so
// a position's result does not depend on how a prompt was cut or on what else is in the step; steps of one token per
// request have a kernel of their own, whose order differs from the portions' (a difference of rounding).
#include "common.cuh"
#include <math.h>
using namespace bspec;

namespace {

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// m <- max(f + m, i), m kept as a pair (leading part, remainder) so that many small f can be added to an m of some units;
// x = f + m_old - m and b = i - m are the logs of the decay and of the input's strength.
__device__ __forceinline__ void advance_maximum(float& m_hi, float& m_lo, float i, float f, float& x, float& b) {
  const float s = __fadd_rn(m_hi, f), z = __fsub_rn(s, m_hi);
  const float err = __fadd_rn(__fadd_rn(__fsub_rn(m_hi, __fsub_rn(s, z)), __fsub_rn(f, z)), m_lo);
  const float hi = __fadd_rn(s, err), lo = __fsub_rn(err, __fsub_rn(hi, s));
  const float d = __fsub_rn(__fsub_rn(i, hi), lo);           // i - (f + m)
  const bool up = d > 0.f;
  m_hi = up ? i : hi;
  m_lo = up ? 0.f : lo;
  x = up ? -d : 0.f;
  b = up ? 0.f : d;
}

// A block of COLS value columns of one head, L lanes per column (8, 16 or 32); lane r of a column keeps rows
// 4 L g + 4 r + e (e < 4, g < NR / 4) of that column of S in registers.  Tokens are staged TT at a time in shared
// memory, the next TT tokens' rows being fetched into registers while the recurrence runs over the current ones.  One
// more warp forms the gates of the next TT tokens meanwhile: exponentials by one lane per token, the running maximum
// (matrix memory) one token after the other.
// The state moves by (exp(x) - 1) S + b k v^T: a head with a long memory has exp(x) within 1e-4 of 1, where a float32
// factor keeps only three digits of what matters.
constexpr int GS_COLS = 16;
constexpr int GS_TT = 16;
constexpr int STATE_SPACE = 0, MATRIX_MEMORY = 1;
constexpr int M_WORDS = 6;           // two records of the running maximum per head: leading part, remainder, position

struct GatedStateArgs {
  const float* q;                    // rows of stride ld_qkv; head h reads columns (h / rep) dim ..
  const float* k;
  const float* v;                    // columns h vdim ..
  long long ld_qkv;
  const float* g0;                   // raw gates: the step size, or the input gate; column h of rows of stride ld_g
  const float* g1;                   // the forget gate (matrix memory)
  long long ld_g;
  const float* p0;                   // per head: bias of the step size / of the input gate
  const float* p1;                   // per head: exp(A_log) / bias of the forget gate
  const float* p2;                   // per head: D (state space)
  float* state;                      // [slot]: S as [H][value columns][dim], then at aux_off what else the form keeps
  long long state_stride, aux_off;
  const float* conv_in;              // state space: the convolution's inputs, its last taps-1 rows go to aux_off
  long long ld_conv;
  const int* qo_indptr;
  const int* state_slots;
  const int* positions;
  float* out;                        // [n, H vdim]
  float* den;                        // [n, H] (matrix memory)
  int H, rep, dim, vdim, channels, taps;
  float q_scale, cap;
};

template <int NR, int L, int KIND>
__global__ void __launch_bounds__(GS_COLS * L + 32)
gated_state_kernel(const GatedStateArgs a) {
  bspec::pdl_prologue_late(KIND == STATE_SPACE ? 74 : 75);
  constexpr int MAIN = GS_COLS * L;
  constexpr int DM = L * NR;                                // rows of S this instance holds (dim <= DM)
  constexpr int VR = (GS_TT * GS_COLS + MAIN - 1) / MAIN;
  static_assert(NR % 4 == 0 && (L == 8 || L == 16 || L == 32) && GS_TT * DM == NR * MAIN, "lanes and rows");
  __shared__ __align__(16) float qs[GS_TT][DM];
  __shared__ __align__(16) float ks[GS_TT][DM];
  __shared__ float vs[GS_TT][GS_COLS];
  __shared__ float gs[2][GS_TT][3];                          // exp(x) - 1, b, exp(-m)
  const int e = blockIdx.z, h = blockIdx.y, H = a.H, dim = a.dim, vdim = a.vdim;
  const int columns = vdim + (KIND == MATRIX_MEMORY ? 1 : 0);        // the last one is n: its value is always 1
  const int t0 = a.qo_indptr[e], nt = a.qo_indptr[e + 1] - t0;
  if (nt <= 0) return;
  float* row = a.state + (size_t)a.state_slots[e] * a.state_stride;
  const bool gate_warp = threadIdx.x >= MAIN;
  const int lane = threadIdx.x & 31;

  // ---- the gate warp
  float m_hi = 0.f, m_lo = 0.f;
  int m_next = 0;                                            // which of the two records is written at the end
  if (KIND == MATRIX_MEMORY && gate_warp) {
    // A head's running maximum is read by all of its blocks and written by one: the record of this portion's first
    // position is read, the other one written, so it does not matter who comes first.
    const float* rec = row + a.aux_off + (size_t)h * M_WORDS;
    const int use = __float_as_int(rec[2]) == a.positions[t0] ? 0 : 1;
    m_hi = rec[3 * use];
    m_lo = rec[3 * use + 1];
    m_next = 1 - use;
  }
  auto gates = [&](int base, int buf) {
    const int cnt = min(GS_TT, nt - base);
    const bool live = lane < cnt;
    const float* at = a.g0 + (size_t)(t0 + base + (live ? lane : 0)) * a.ld_g + h;
    if constexpr (KIND == STATE_SPACE) {
      const float dt = softplus_f(at[0] + a.p0[h]);
      if (live) {
        gs[buf][lane][0] = expm1f(-a.p1[h] * dt);
        gs[buf][lane][1] = dt;
      }
    } else {
      const float raw_f = a.g1[(size_t)(t0 + base + (live ? lane : 0)) * a.ld_g + h];
      const float i_log = a.cap * tanhf((at[0] + a.p0[h]) / a.cap);
      const float f_log = -softplus_f(-a.cap * tanhf((raw_f + a.p1[h]) / a.cap));
      float x = 0.f, b_log = 0.f, m = 0.f;
#pragma unroll
      for (int t = 0; t < GS_TT; ++t) {
        const float it = __shfl_sync(0xffffffffu, i_log, t), ft = __shfl_sync(0xffffffffu, f_log, t);
        if (t >= cnt) break;
        float xt, bt;
        advance_maximum(m_hi, m_lo, it, ft, xt, bt);
        if (lane == t) {
          x = xt;
          b_log = bt;
          m = m_hi;
        }
      }
      if (live) {
        gs[buf][lane][0] = expm1f(x);
        gs[buf][lane][1] = expf(b_log);
        gs[buf][lane][2] = expf(-m);
      }
    }
  };

  // ---- the other warps
  const int col = threadIdx.x / L, r = threadIdx.x % L;
  const int j = blockIdx.x * GS_COLS + col;                  // value column of the head
  const bool live = !gate_warp && j < columns;
  float* sp = row + ((size_t)h * columns + (live ? j : 0)) * dim;
  float qn[NR], kn[NR], vn[VR];
  auto fetch = [&](int base) {
    const int cnt = min(GS_TT, nt - base);
#pragma unroll
    for (int u = 0; u < NR; ++u) {
      const int x = threadIdx.x + MAIN * u;
      const int tt = x / DM, i = x % DM;                     // tt is the same for a whole warp (DM >= 32)
      if (tt >= cnt) break;
      const bool ok = i < dim;
      const size_t at = (size_t)(t0 + base + tt) * a.ld_qkv + (size_t)(h / a.rep) * dim + (ok ? i : 0);
      qn[u] = ok ? a.q[at] : 0.f;
      kn[u] = ok ? a.k[at] : 0.f;
    }
#pragma unroll
    for (int u = 0; u < VR; ++u) {
      const int x = threadIdx.x + MAIN * u;
      const int tt = x / GS_COLS, c = x % GS_COLS;
      const int jj = blockIdx.x * GS_COLS + c;
      const bool in = x < GS_TT * GS_COLS && tt < cnt;
      vn[u] = in && jj < vdim ? a.v[(size_t)(t0 + base + tt) * a.ld_qkv + (size_t)h * vdim + jj] : (jj == vdim ? 1.f : 0.f);
    }
  };
  float s[NR];
  const bool vec = (dim & 3) == 0 && (reinterpret_cast<uintptr_t>(sp) & 15) == 0;
  if (gate_warp) {
    gates(0, 0);
  } else {
    fetch(0);
    if (vec) {
#pragma unroll
      for (int g = 0; g < NR / 4; ++g) {
        const int i = 4 * L * g + 4 * r;
        const float4 v4 = (live && i < dim) ? *reinterpret_cast<const float4*>(sp + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        s[4 * g] = v4.x, s[4 * g + 1] = v4.y, s[4 * g + 2] = v4.z, s[4 * g + 3] = v4.w;
      }
    } else {
#pragma unroll
      for (int w = 0; w < NR; ++w) {
        const int i = 4 * L * (w >> 2) + 4 * r + (w & 3);
        s[w] = (live && i < dim) ? sp[i] : 0.f;
      }
    }
  }
  if (KIND == STATE_SPACE && a.taps > 1) {
    // the convolution's inputs move on: slot u holds the input at index nt + u - (taps - 1) of this portion, or what an
    // older slot held; ascending, so that a slot is read before it is overwritten.  The request's blocks share the
    // channels (a thread moves all slots of its channel).
    float* tail = row + a.aux_off;
    const int C = a.channels, share = blockIdx.y * gridDim.x + blockIdx.x, shares = gridDim.y * gridDim.x;
    for (int c = share * (MAIN + 32) + threadIdx.x; c < C; c += shares * (MAIN + 32))
      for (int u = 0; u < a.taps - 1; ++u) {
        const int rel = nt + u - (a.taps - 1);
        tail[(size_t)u * C + c] = rel >= 0 ? a.conv_in[(size_t)(t0 + rel) * a.ld_conv + c] : tail[(size_t)(u + nt) * C + c];
      }
  }
  const float skip = KIND == STATE_SPACE ? a.p2[h] : 0.f;
  auto write = [&](int t, int tt, int buf, float acc) {      // the token's result for this thread's column
    if (KIND == MATRIX_MEMORY && j == vdim)
      a.den[(size_t)t * H + h] = fmaxf(fabsf(acc), gs[buf][tt][2]) + 1e-6f;
    else
      a.out[((size_t)t * H + h) * vdim + j] = KIND == STATE_SPACE ? __fmaf_rn(skip, vs[tt][col], acc) : acc;
  };
  int buf = 0;
  for (int base = 0; base < nt; base += GS_TT, buf ^= 1) {
    const int cnt = min(GS_TT, nt - base);
    __syncthreads();
    if (!gate_warp) {
#pragma unroll
      for (int u = 0; u < NR; ++u) {                         // rows of tokens beyond cnt are never read
        const int x = threadIdx.x + MAIN * u;
        if (x / DM >= cnt) break;
        qs[x / DM][x % DM] = qn[u] * a.q_scale;
        ks[x / DM][x % DM] = kn[u];
      }
#pragma unroll
      for (int u = 0; u < VR; ++u) {
        const int x = threadIdx.x + MAIN * u;
        if (x < GS_TT * GS_COLS && x / GS_COLS < cnt) vs[x / GS_COLS][x % GS_COLS] = vn[u];
      }
    }
    __syncthreads();
    if (gate_warp) {
      if (base + GS_TT < nt) gates(base + GS_TT, buf ^ 1);
      continue;
    }
    if (base + GS_TT < nt) fetch(base + GS_TT);
    int tt = 0;
    for (; tt + 4 <= cnt; tt += 4) {
      float acc[4] = {0.f, 0.f, 0.f, 0.f}, vj[4], em1[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        vj[u] = __fmul_rn(gs[buf][tt + u][1], vs[tt + u][col]);
        em1[u] = gs[buf][tt + u][0];
      }
#pragma unroll
      for (int g = 0; g < NR / 4; ++g) {
        float4 k4[4], q4[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          k4[u] = *reinterpret_cast<const float4*>(&ks[tt + u][4 * L * g + 4 * r]);
          q4[u] = *reinterpret_cast<const float4*>(&qs[tt + u][4 * L * g + 4 * r]);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float kk[4] = {k4[u].x, k4[u].y, k4[u].z, k4[u].w}, qq[4] = {q4[u].x, q4[u].y, q4[u].z, q4[u].w};
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            s[4 * g + c] = __fadd_rn(s[4 * g + c], __fmaf_rn(em1[u], s[4 * g + c], __fmul_rn(kk[c], vj[u])));
            acc[u] = __fmaf_rn(s[4 * g + c], qq[c], acc[u]);
          }
        }
      }
#pragma unroll
      for (int o = 1; o < L; o <<= 1)
#pragma unroll
        for (int u = 0; u < 4; ++u) acc[u] += __shfl_xor_sync(0xffffffffu, acc[u], o);
      const float mine = r == 0 ? acc[0] : (r == 1 ? acc[1] : (r == 2 ? acc[2] : acc[3]));
      if (live && r < 4) write(t0 + base + tt + r, tt + r, buf, mine);
    }
    for (; tt < cnt; ++tt) {
      const float vj = __fmul_rn(gs[buf][tt][1], vs[tt][col]), em1 = gs[buf][tt][0];
      float acc = 0.f;
#pragma unroll
      for (int g = 0; g < NR / 4; ++g) {
        const float4 k4 = *reinterpret_cast<const float4*>(&ks[tt][4 * L * g + 4 * r]);
        const float4 q4 = *reinterpret_cast<const float4*>(&qs[tt][4 * L * g + 4 * r]);
        const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          s[4 * g + c] = __fadd_rn(s[4 * g + c], __fmaf_rn(em1, s[4 * g + c], __fmul_rn(kk[c], vj)));
          acc = __fmaf_rn(s[4 * g + c], qq[c], acc);
        }
      }
#pragma unroll
      for (int o = 1; o < L; o <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
      if (live && r == 0) write(t0 + base + tt, tt, buf, acc);
    }
  }
  bspec::pdl_launch_dependents();
  if (KIND == MATRIX_MEMORY && gate_warp && blockIdx.x == 0 && lane == 0) {
    float* rec = row + a.aux_off + (size_t)h * M_WORDS + 3 * m_next;
    rec[0] = m_hi;
    rec[1] = m_lo;
    rec[2] = __int_as_float(a.positions[t0] + nt);
  }
  if (live && vec) {
#pragma unroll
    for (int g = 0; g < NR / 4; ++g) {
      const int i = 4 * L * g + 4 * r;
      if (i < dim) *reinterpret_cast<float4*>(sp + i) = make_float4(s[4 * g], s[4 * g + 1], s[4 * g + 2], s[4 * g + 3]);
    }
  } else if (live) {
#pragma unroll
    for (int w = 0; w < NR; ++w) {
      const int i = 4 * L * (w >> 2) + 4 * r + (w & 3);
      if (i < dim) sp[i] = s[w];
    }
  }
}

// A step in which every portion is one token (decoding): bound by reading and writing the state once.  Nothing is staged:
// LPC lanes share a value column of QPL x 4 LPC rows, a warp takes several columns at a time whose loads are all in flight
// together, and every warp forms its head's gates itself.  The state was last written by an earlier step, so its loads are
// issued before the wait on the kernel before this one (which writes q, k, v and the gates).
constexpr int GD_WARPS = 4;

template <int KIND, int LPC, int QPL, int CPL>             // CPL: columns per lane group
__global__ void __launch_bounds__(GD_WARPS * 32)
gated_state_decode_kernel(const GatedStateArgs a) {
  const unsigned long long t_trace = bspec::g_trace_buf != nullptr ? bspec::global_timer() : 0ull;
  bspec::pdl_launch_dependents();
  constexpr int GROUPS = 32 / LPC;                           // lane groups of a warp
  const int e = blockIdx.z, h = blockIdx.y, H = a.H, dim = a.dim, vdim = a.vdim;
  const int columns = vdim + (KIND == MATRIX_MEMORY ? 1 : 0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, grp = lane / LPC, r = lane % LPC;
  const int t = a.qo_indptr[e];
  float* row = a.state + (size_t)a.state_slots[e] * a.state_stride;
  const int j0 = (blockIdx.x * GD_WARPS + warp) * GROUPS * CPL + grp;          // the group's columns: j0, j0 + GROUPS, ...
  float4 s[CPL][QPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    const int j = j0 + c * GROUPS;
    const float* sp = row + ((size_t)h * columns + j) * dim;
#pragma unroll
    for (int k = 0; k < QPL; ++k) {
      const int i = 4 * (r + k * LPC);
      s[c][k] = j < columns && i < dim ? *reinterpret_cast<const float4*>(sp + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  bspec::pdl_wait();
  bspec::trace_record(KIND == STATE_SPACE ? 74 : 75, t_trace);
  float4 q[QPL], k4[QPL];
  const size_t at = (size_t)t * a.ld_qkv + (size_t)(h / a.rep) * dim;
#pragma unroll
  for (int k = 0; k < QPL; ++k) {
    const int i = 4 * (r + k * LPC);
    q[k] = k4[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < dim) {
      q[k] = *reinterpret_cast<const float4*>(a.q + at + i);
      k4[k] = *reinterpret_cast<const float4*>(a.k + at + i);
    }
    q[k].x *= a.q_scale; q[k].y *= a.q_scale; q[k].z *= a.q_scale; q[k].w *= a.q_scale;
  }
  float v[CPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    const int j = j0 + c * GROUPS;
    v[c] = j < vdim ? a.v[(size_t)t * a.ld_qkv + (size_t)h * vdim + j] : (j == vdim ? 1.f : 0.f);
  }
  float em1, b, exp_m = 0.f;
  const float raw = a.g0[(size_t)t * a.ld_g + h];
  if constexpr (KIND == STATE_SPACE) {
    b = softplus_f(raw + a.p0[h]);
    em1 = expm1f(-a.p1[h] * b);
  } else {
    const float* rec = row + a.aux_off + (size_t)h * M_WORDS;
    const int pos = a.positions[t], use = __float_as_int(rec[2]) == pos ? 0 : 1;
    float m_hi = rec[3 * use], m_lo = rec[3 * use + 1], x, b_log;
    const float i_log = a.cap * tanhf((raw + a.p0[h]) / a.cap);
    const float f_log = -softplus_f(-a.cap * tanhf((a.g1[(size_t)t * a.ld_g + h] + a.p1[h]) / a.cap));
    advance_maximum(m_hi, m_lo, i_log, f_log, x, b_log);
    em1 = expm1f(x);
    b = expf(b_log);
    exp_m = expf(-m_hi);
    if (blockIdx.x == 0 && threadIdx.x == 0) {               // the other record: nobody reads it as this position's
      float* to = row + a.aux_off + (size_t)h * M_WORDS + 3 * (1 - use);
      to[0] = m_hi;
      to[1] = m_lo;
      to[2] = __int_as_float(pos + 1);
    }
  }
  if (KIND == STATE_SPACE && a.taps > 1) {                   // the convolution's inputs move on by one
    float* tail = row + a.aux_off;
    const int C = a.channels, share = blockIdx.y * gridDim.x + blockIdx.x, shares = gridDim.y * gridDim.x;
    for (int c = share * (GD_WARPS * 32) + threadIdx.x; c < C; c += shares * (GD_WARPS * 32)) {
      for (int u = 0; u < a.taps - 2; ++u) tail[(size_t)u * C + c] = tail[(size_t)(u + 1) * C + c];
      tail[(size_t)(a.taps - 2) * C + c] = a.conv_in[(size_t)t * a.ld_conv + c];
    }
  }
  float acc[CPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    const int j = j0 + c * GROUPS;
    const float bv = __fmul_rn(b, v[c]);
    float* sp = row + ((size_t)h * columns + j) * dim;
    acc[c] = 0.f;
#pragma unroll
    for (int k = 0; k < QPL; ++k) {
      float4& x = s[c][k];
      x.x = __fadd_rn(x.x, __fmaf_rn(em1, x.x, __fmul_rn(k4[k].x, bv)));
      x.y = __fadd_rn(x.y, __fmaf_rn(em1, x.y, __fmul_rn(k4[k].y, bv)));
      x.z = __fadd_rn(x.z, __fmaf_rn(em1, x.z, __fmul_rn(k4[k].z, bv)));
      x.w = __fadd_rn(x.w, __fmaf_rn(em1, x.w, __fmul_rn(k4[k].w, bv)));
      acc[c] = __fmaf_rn(x.x, q[k].x, acc[c]);
      acc[c] = __fmaf_rn(x.y, q[k].y, acc[c]);
      acc[c] = __fmaf_rn(x.z, q[k].z, acc[c]);
      acc[c] = __fmaf_rn(x.w, q[k].w, acc[c]);
      const int i = 4 * (r + k * LPC);
      if (j < columns && i < dim) *reinterpret_cast<float4*>(sp + i) = x;
    }
  }
#pragma unroll
  for (int o = 1; o < LPC; o <<= 1)
#pragma unroll
    for (int c = 0; c < CPL; ++c) acc[c] += __shfl_xor_sync(0xffffffffu, acc[c], o);
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    const int j = j0 + c * GROUPS;
    if (r != c % LPC || j >= columns) continue;
    if (KIND == MATRIX_MEMORY && j == vdim) a.den[(size_t)t * H + h] = fmaxf(fabsf(acc[c]), exp_m) + 1e-6f;
    else a.out[((size_t)t * H + h) * vdim + j] = KIND == STATE_SPACE ? __fmaf_rn(a.p2[h], v[c], acc[c]) : acc[c];
  }
}

template <int KIND>
int launch_gated_state(const GatedStateArgs& a, int n_entries, int max_q_len, cudaStream_t stream) {
  if (n_entries <= 0) return 0;
  if (a.dim <= 0 || a.dim > 256 || a.vdim <= 0 || a.H <= 0 || a.H > 65535 || a.rep <= 0 || a.H % a.rep || n_entries > 65535 ||
      a.taps < 1 || a.channels < 0)
    return (int)cudaErrorInvalidValue;
  const int columns = a.vdim + (KIND == MATRIX_MEMORY ? 1 : 0);
  const uintptr_t bases = reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.k) | reinterpret_cast<uintptr_t>(a.state);
  if (max_q_len == 1 && a.dim % 4 == 0 && a.ld_qkv % 4 == 0 && a.state_stride % 4 == 0 && (bases & 15) == 0) {
#define LD(LPC, QPL, CPL)                                                                                          \
  BSPEC_LAUNCH((gated_state_decode_kernel<KIND, LPC, QPL, CPL>),                                                   \
               dim3((columns + GD_WARPS * (32 / LPC) * CPL - 1) / (GD_WARPS * (32 / LPC) * CPL), a.H, n_entries),  \
               GD_WARPS * 32, 0, stream, a)
    if (a.dim <= 32) LD(8, 1, 4);
    else if (a.dim <= 64) LD(16, 1, 4);
    else if (a.dim <= 128) LD(32, 1, 8);
    else LD(32, 2, 4);
#undef LD
    return BSPEC_LAUNCH_CHECK();
  }
  const dim3 grid((columns + GS_COLS - 1) / GS_COLS, a.H, n_entries);
  // Lanes per column, by the sizes alone: fewer lanes share more of what they read from shared memory, more lanes have a
  // shorter chain per token.  (Measured on prompts of 2,048 tokens, 128 to 4,096 blocks, 8 / 16 / 32 lanes: 16 lanes are
  // best for the state space from 128 blocks up, 8 for the matrix memory.)
  constexpr bool WIDE = KIND == STATE_SPACE;
#define LG(NR, L) \
  BSPEC_LAUNCH_SERIALIZED((gated_state_kernel<NR, L, KIND>), grid, GS_COLS * (L) + 32, 0, stream, a)
  if (a.dim <= 32) LG(4, 8);
  else if (a.dim <= 64) LG(WIDE ? 4 : 8, WIDE ? 16 : 8);
  else if (a.dim <= 128) LG(WIDE ? 8 : 16, WIDE ? 16 : 8);
  else LG(16, 16);
#undef LG
  return BSPEC_LAUNCH_CHECK();
}
}  // namespace

// xbc [n, >= H vdim + 2 groups dim] float32 rows of stride ld: [v: H vdim | k: groups dim | q: groups dim] after the
// convolution; conv_in rows of stride ld_in: the same columns before it, and the raw step sizes at dt (column h).
// rate [H] = exp(A_log).  State row: [S as [H][vdim][dim] | at tail_off the last taps-1 rows of conv_in's columns].
BSPEC_API int bspec_state_space(const float* xbc, long long ld, const float* conv_in, const float* dt, long long ld_in,
                                const float* dt_bias, const float* rate, const float* skip, float* state,
                                long long state_stride, long long tail_off, const int* qo_indptr, const int* state_slots,
                                const int* positions, float* out, int n_entries, int max_q_len, int H, int groups,
                                int dim, int vdim, int taps, cudaStream_t stream) {
  if (groups <= 0 || H % groups) return (int)cudaErrorInvalidValue;
  GatedStateArgs a = {};
  a.v = xbc; a.k = xbc + (size_t)H * vdim; a.q = a.k + (size_t)groups * dim; a.ld_qkv = ld;
  a.g0 = dt; a.ld_g = ld_in; a.p0 = dt_bias; a.p1 = rate; a.p2 = skip;
  a.state = state; a.state_stride = state_stride; a.aux_off = tail_off; a.conv_in = conv_in; a.ld_conv = ld_in;
  a.qo_indptr = qo_indptr; a.state_slots = state_slots; a.positions = positions; a.out = out;
  a.H = H; a.rep = H / groups; a.dim = dim; a.vdim = vdim; a.channels = H * vdim + 2 * groups * dim; a.taps = taps;
  a.q_scale = 1.f;
  return launch_gated_state<STATE_SPACE>(a, n_entries, max_q_len, stream);
}

// proj [n, ld] float32: columns q and k (H dim each), v (H vdim), and the raw gates i and f (H each) at their offsets.
// State row: [S as [H][vdim + 1][dim], column vdim being n | at m_off the running maximum's records [H][6]].
BSPEC_API int bspec_matrix_memory(const float* proj, long long ld, int q_off, int k_off, int v_off, int i_off, int f_off,
                                  const float* i_bias, const float* f_bias, float cap, float q_scale, float* state,
                                  long long state_stride, long long m_off, const int* qo_indptr, const int* state_slots,
                                  const int* positions, float* out, float* den, int n_entries, int max_q_len, int H,
                                  int dim, int vdim, cudaStream_t stream) {
  if (!(cap > 0.f)) return (int)cudaErrorInvalidValue;
  GatedStateArgs a = {};
  a.q = proj + q_off; a.k = proj + k_off; a.v = proj + v_off; a.ld_qkv = ld;
  a.g0 = proj + i_off; a.g1 = proj + f_off; a.ld_g = ld; a.p0 = i_bias; a.p1 = f_bias;
  a.state = state; a.state_stride = state_stride; a.aux_off = m_off;
  a.qo_indptr = qo_indptr; a.state_slots = state_slots; a.positions = positions; a.out = out; a.den = den;
  a.H = H; a.rep = 1; a.dim = dim; a.vdim = vdim; a.taps = 1; a.q_scale = q_scale; a.cap = cap;
  return launch_gated_state<MATRIX_MEMORY>(a, n_entries, max_q_len, stream);
}

BSPEC_DEFINE_TRACE_SETTER(bspec_trace_set_gated_states)
