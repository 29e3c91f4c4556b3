// How a sublayer's result joins the residual stream when it is normed on its way, and averages over depth.
//
// branch_join, one block per row; every part of it is optional:
//   y  = delta,  or the pair  delta / rms(delta) * wa + delta_b / rms(delta_b) * wb
//   x  = src + extra + y,  or with a weight ``post``:  src + extra + y / rms(y) * post      (``extra``: a second branch)
//   hist[slot] = x                                                      (``store``)
//   x  = sum_{j < slot} coef[j] hist[j] + coef[slot] x                  (``coef``: the average over the layers so far)
//   dst = x
//   out = x / rms(x) * norm_w,  or the cast of x without a weight
// rms(v) = sqrt(mean(v^2) + eps).  All arithmetic is float32; ``out`` is rounded once.  ``rows``: block i works on row
// rows[i] of src, delta and hist and writes row i of dst and out (the rows that go to the head).
// A row stays in registers from its first read to its last write (four columns per thread and pass); the layers'
// history is read while the branch's sum of squares is still being formed.  Widths that are no multiple of 4, or
// above 16,384, keep the row in shared memory instead.
#include "common.cuh"
using namespace bspec;

namespace {

struct JoinArgs {
  const float* src;          // [*, d] or null (zeros)
  float* dst;                // [n, d] or null; may be src
  const int* rows;           // [n] or null
  const void* delta;         // [*, d] or null
  const void* delta_b;       // the second of a pair, or null
  const void* extra;         // [*, d] another branch, added as it is (of delta's type), or null
  const float* wa;           // [d] weights of the pair
  const float* wb;
  const float* post;         // [d] or null
  float* hist;               // [slots][*, d] or null
  const float* coef;         // [slot + 1] or null
  const float* norm_w;       // [d] or null
  void* out;                 // [n, d] or null
  long long hist_stride;     // elements from one slot to the next
  long long n_src;           // rows of src, delta and hist (checked build)
  int slot, store, d;
  float branch_eps, eps;
};

template <typename T> __device__ __forceinline__ void load4(const T* p, float (&f)[4]);
template <> __device__ __forceinline__ void load4<float>(const float* p, float (&f)[4]) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
template <> __device__ __forceinline__ void load4<__nv_bfloat16>(const __nv_bfloat16* p, float (&f)[4]) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&v.x), b = *reinterpret_cast<const __nv_bfloat162*>(&v.y);
  f[0] = __low2float(a); f[1] = __high2float(a); f[2] = __low2float(b); f[3] = __high2float(b);
}
template <typename T> __device__ __forceinline__ void store4(T* p, const float (&f)[4]);
template <> __device__ __forceinline__ void store4<float>(float* p, const float (&f)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, const float (&f)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
  uint2 v;
  v.x = *reinterpret_cast<const uint32_t*>(&a);
  v.y = *reinterpret_cast<const uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = v;
}

// Block-wide sums with a fixed tree; every call of a kernel has 32 floats of its own, so one barrier is enough.
__device__ __forceinline__ float sum_once(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  return warp_sum(lane < nwarps ? scratch[lane] : 0.f);
}
__device__ __forceinline__ void sum_once2(float& a, float& b, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  if (lane == 0) { scratch[warp] = a; scratch[32 + warp] = b; }
  __syncthreads();
  a = warp_sum(lane < nwarps ? scratch[lane] : 0.f);
  b = warp_sum(lane < nwarps ? scratch[32 + lane] : 0.f);
}

template <typename TD, typename TO, int VPT, bool PAIR, bool DEPTH>
__global__ void branch_join_kernel(const JoinArgs a) {
  bspec::pdl_prologue(73);
  __shared__ float scratch[128];
  const int d = a.d;
  long long row = a.rows != nullptr ? a.rows[blockIdx.x] : (long long)blockIdx.x;
  if (!bspec::in_range(row, a.n_src, 115)) return;
  const size_t base = (size_t)row * d, obase = (size_t)blockIdx.x * d;
  float x[VPT][4], y[VPT][4], z[PAIR ? VPT : 1][4], h[DEPTH ? VPT : 1][4];
  float sa = 0.f, sb = 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = 4 * (threadIdx.x + k * blockDim.x);
#pragma unroll
    for (int c = 0; c < 4; ++c) x[k][c] = y[k][c] = h[DEPTH ? k : 0][c] = 0.f;
    if (i < d) {
      if (a.src != nullptr) load4<float>(a.src + base + i, x[k]);
      if (a.extra != nullptr) {
        float v[4];
        load4<TD>(reinterpret_cast<const TD*>(a.extra) + base + i, v);
#pragma unroll
        for (int c = 0; c < 4; ++c) x[k][c] += v[c];
      }
      if (a.delta != nullptr) load4<TD>(reinterpret_cast<const TD*>(a.delta) + base + i, y[k]);
      if (PAIR) load4<TD>(reinterpret_cast<const TD*>(a.delta_b) + base + i, z[PAIR ? k : 0]);
    }
  }
  if (DEPTH) {
#pragma unroll 2
    for (int j = 0; j < a.slot; ++j) {
      const float w = a.coef[j];
      const float* hp = a.hist + (size_t)j * a.hist_stride + base;
#pragma unroll
      for (int k = 0; k < VPT; ++k) {
        const int i = 4 * (threadIdx.x + k * blockDim.x);
        if (i < d) {
          float v[4];
          load4<float>(hp + i, v);
#pragma unroll
          for (int c = 0; c < 4; ++c) h[DEPTH ? k : 0][c] += w * v[c];
        }
      }
    }
  }
  if (PAIR) {
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = 4 * (threadIdx.x + k * blockDim.x);
      if (i < d)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          sa += y[k][c] * y[k][c];
          sb += z[PAIR ? k : 0][c] * z[PAIR ? k : 0][c];
        }
    }
    sum_once2(sa, sb, scratch);
    const float ra = 1.f / sqrtf(sa / (float)d + a.branch_eps), rb = 1.f / sqrtf(sb / (float)d + a.branch_eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = 4 * (threadIdx.x + k * blockDim.x);
      if (i < d) {
        float wa[4], wb[4];
        load4<float>(a.wa + i, wa);
        load4<float>(a.wb + i, wb);
#pragma unroll
        for (int c = 0; c < 4; ++c)
          y[k][c] = y[k][c] * ra * wa[c] + z[PAIR ? k : 0][c] * rb * wb[c];
      }
    }
  }
  if (a.post != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k)
#pragma unroll
      for (int c = 0; c < 4; ++c) ss += y[k][c] * y[k][c];           // zeros beyond the row
    const float r = 1.f / sqrtf(sum_once(ss, scratch + 64) / (float)d + a.branch_eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = 4 * (threadIdx.x + k * blockDim.x);
      if (i < d) {
        float w[4];
        load4<float>(a.post + i, w);
#pragma unroll
        for (int c = 0; c < 4; ++c) y[k][c] = y[k][c] * r * w[c];
      }
    }
  }
  const float own = DEPTH ? a.coef[a.slot] : 1.f;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = 4 * (threadIdx.x + k * blockDim.x);
    if (i < d) {
#pragma unroll
      for (int c = 0; c < 4; ++c) x[k][c] += y[k][c];
      if (a.store) store4<float>(a.hist + (size_t)a.slot * a.hist_stride + base + i, x[k]);
      if (DEPTH)
#pragma unroll
        for (int c = 0; c < 4; ++c) x[k][c] = h[DEPTH ? k : 0][c] + own * x[k][c];
      if (a.dst != nullptr) store4<float>(a.dst + obase + i, x[k]);
#pragma unroll
      for (int c = 0; c < 4; ++c) ss += x[k][c] * x[k][c];
    }
  }
  if (a.out == nullptr) return;
  const float r = a.norm_w != nullptr ? 1.f / sqrtf(sum_once(ss, scratch + 96) / (float)d + a.eps) : 1.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = 4 * (threadIdx.x + k * blockDim.x);
    if (i < d) {
      float w[4] = {1.f, 1.f, 1.f, 1.f}, o[4];
      if (a.norm_w != nullptr) load4<float>(a.norm_w + i, w);
#pragma unroll
      for (int c = 0; c < 4; ++c) o[c] = x[k][c] * r * w[c];
      store4<TO>(reinterpret_cast<TO*>(a.out) + obase + i, o);
    }
  }
}

// Any width: the row in shared memory, one column per thread and pass.
template <typename TD, typename TO>
__global__ void branch_join_any_kernel(const JoinArgs a) {
  bspec::pdl_prologue(73);
  extern __shared__ float ys[];                       // [d] the branch, then the new row
  __shared__ float scratch[128];
  const int d = a.d;
  long long row = a.rows != nullptr ? a.rows[blockIdx.x] : (long long)blockIdx.x;
  if (!bspec::in_range(row, a.n_src, 115)) return;
  const size_t base = (size_t)row * d, obase = (size_t)blockIdx.x * d;
  const TD* da = reinterpret_cast<const TD*>(a.delta);
  const TD* db = reinterpret_cast<const TD*>(a.delta_b);
  float sa = 0.f, sb = 0.f;
  if (db != nullptr) {
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
      const float u = to_f32(da[base + i]), v = to_f32(db[base + i]);
      sa += u * u;
      sb += v * v;
    }
    sum_once2(sa, sb, scratch);
  }
  const float ra = 1.f / sqrtf(sa / (float)d + a.branch_eps), rb = 1.f / sqrtf(sb / (float)d + a.branch_eps);
  float ss = 0.f;
  for (int i = threadIdx.x; i < d; i += blockDim.x) {
    float y = da != nullptr ? to_f32(da[base + i]) : 0.f;
    if (db != nullptr) y = y * ra * a.wa[i] + to_f32(db[base + i]) * rb * a.wb[i];
    ys[i] = y;                                        // a thread reads back only its own columns
    ss += y * y;
  }
  const float rp = a.post != nullptr ? 1.f / sqrtf(sum_once(ss, scratch + 64) / (float)d + a.branch_eps) : 1.f;
  ss = 0.f;
  for (int i = threadIdx.x; i < d; i += blockDim.x) {
    float x = a.src != nullptr ? a.src[base + i] : 0.f;
    if (a.extra != nullptr) x += to_f32(reinterpret_cast<const TD*>(a.extra)[base + i]);
    x += ys[i] * rp * (a.post != nullptr ? a.post[i] : 1.f);
    if (a.store) a.hist[(size_t)a.slot * a.hist_stride + base + i] = x;
    if (a.coef != nullptr) {
      float h = 0.f;
      for (int j = 0; j < a.slot; ++j) h += a.coef[j] * a.hist[(size_t)j * a.hist_stride + base + i];
      x = h + a.coef[a.slot] * x;
    }
    if (a.dst != nullptr) a.dst[obase + i] = x;
    ys[i] = x;
    ss += x * x;
  }
  if (a.out == nullptr) return;
  const float r = a.norm_w != nullptr ? 1.f / sqrtf(sum_once(ss, scratch + 96) / (float)d + a.eps) : 1.f;
  for (int i = threadIdx.x; i < d; i += blockDim.x)
    reinterpret_cast<TO*>(a.out)[obase + i] = from_f32<TO>(ys[i] * r * (a.norm_w != nullptr ? a.norm_w[i] : 1.f));
}

template <typename TD, typename TO>
int launch_join(const JoinArgs& a, int n, cudaStream_t stream) {
  const int d = a.d;
  if (d % 4 == 0 && d <= 4 * 4 * 1024) {
    const int quads = d / 4;
    int threads = quads >= 1024 ? 1024 : ((quads + 31) / 32) * 32;
    // Many rows: four quads per thread, so that a thread has more loads in flight and several rows share an SM.
    // Only for bfloat16 output: in float32 a row's sums keep one order, whatever else is in the step.
    if (sizeof(TO) == 2 && n >= 512 && quads >= 128) threads = (((quads + 3) / 4 + 31) / 32) * 32;
    if (threads > 1024) threads = 1024;
    const int vpt = (quads + threads - 1) / threads;
#define LJP(V, P)                                                                                              \
  do {                                                                                                         \
    if (a.coef != nullptr) BSPEC_LAUNCH((branch_join_kernel<TD, TO, V, P, true>), n, threads, 0, stream, a);     \
    else BSPEC_LAUNCH((branch_join_kernel<TD, TO, V, P, false>), n, threads, 0, stream, a);                      \
  } while (0)
#define LJ(V) do { if (a.delta_b != nullptr) LJP(V, true); else LJP(V, false); } while (0)
    if (vpt <= 1) LJ(1); else if (vpt <= 2) LJ(2); else LJ(4);
#undef LJ
#undef LJP
    return BSPEC_LAUNCH_CHECK();
  }
  const size_t smem = (size_t)d * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(branch_join_any_kernel<TD, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  const int threads = d >= 2048 ? 512 : (d >= 512 ? 256 : 128);
  BSPEC_LAUNCH((branch_join_any_kernel<TD, TO>), n, threads, smem, stream, a);
  return BSPEC_LAUNCH_CHECK();
}
}  // namespace

// Every pointer but the sizes may be null where the comment at the top calls its part optional.
BSPEC_API int bspec_branch_join(const float* src, float* dst, const int* rows, const void* delta, const void* delta_b,
                                const void* extra, int delta_dtype, const float* wa, const float* wb, const float* post,
                                float branch_eps, float* hist, long long hist_stride, int slot, int store,
                                const float* coef, const float* norm_w, float eps, void* out, int out_dtype, int n,
                                long long n_src, int d, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (d <= 0 || slot < 0 || ((store || coef != nullptr) && hist == nullptr) ||
      (delta_b != nullptr && (delta == nullptr || wa == nullptr || wb == nullptr)) ||
      ((post != nullptr || extra != nullptr) && delta == nullptr))
    return (int)cudaErrorInvalidValue;
  JoinArgs a;
  a.src = src; a.dst = dst; a.rows = rows; a.delta = delta; a.delta_b = delta_b; a.extra = extra; a.wa = wa; a.wb = wb; a.post = post;
  a.hist = hist; a.coef = coef; a.norm_w = norm_w; a.out = out; a.hist_stride = hist_stride; a.n_src = n_src;
  a.slot = slot; a.store = store; a.d = d; a.branch_eps = branch_eps; a.eps = eps;
  if (delta_dtype == BSPEC_F32)
    return out_dtype == BSPEC_F32 ? launch_join<float, float>(a, n, stream)
                                  : launch_join<float, __nv_bfloat16>(a, n, stream);
  return out_dtype == BSPEC_F32 ? launch_join<__nv_bfloat16, float>(a, n, stream)
                                : launch_join<__nv_bfloat16, __nv_bfloat16>(a, n, stream);
}

BSPEC_DEFINE_TRACE_SETTER(bspec_trace_set_joins)
BSPEC_DEFINE_BOUNDS_REPORT(bspec_bounds_report_joins)
