// One step of a residual stream between two sublayers, in one kernel:
//
//   X     = x[row] + mult * y[row]                       what the sublayer before has made of the stream (y optional)
//   keep[row] = X                                        if a later layer will ask for it
//   x'    = dw[0] E[row] + sum_k dw[k] P[k - 1][row] (k = 1 .. n) + dw[n + 1] X     with depth weights dw, else x' = X
//   x_out[row] = x'                                      the stream for the sublayer after (may be x itself)
//   out   = norm(x')                                     layer norm (variance: the mean of the squared deviations), RMS norm
//                                                        or none; weight, and optionally a bias, rounded once to the output type
//
// The depth average: E are the rows the embedding left and P[k] the kept results of the layers before, so a layer hands on a
// weighted sum of everything the stream has been.  All arithmetic is float32 in an order that depends on the row alone:
// the terms of the average are added one after the other, E first.  A block per row, the row in registers; four terms of
// the average are asked for before the first is added.  `rows` selects rows (the final norm on the wanted rows only).
#include "common.cuh"

namespace {

constexpr int DEPTH_THREADS = 1024;      // at most; a row of W values takes W / VEC threads if that is fewer

template <int VEC> struct Values { float v[VEC]; };

template <int VEC> __device__ __forceinline__ Values<VEC> depth_load(const float* p) {
  Values<VEC> r;
  if constexpr (VEC == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w;
  } else {
    r.v[0] = p[0];
  }
  return r;
}
template <int VEC> __device__ __forceinline__ Values<VEC> depth_load(const __nv_bfloat16* p) {
  Values<VEC> r;
  if constexpr (VEC == 4) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
    r.v[0] = a.x; r.v[1] = a.y; r.v[2] = b.x; r.v[3] = b.y;
  } else {
    r.v[0] = __bfloat162float(p[0]);
  }
  return r;
}
template <int VEC> __device__ __forceinline__ void depth_store(float* p, const Values<VEC>& x) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(x.v[0], x.v[1], x.v[2], x.v[3]);
  else p[0] = x.v[0];
}
template <int VEC> __device__ __forceinline__ void depth_store(__nv_bfloat16* p, const Values<VEC>& x) {
  if constexpr (VEC == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(x.v[0], x.v[1]), b = __floats2bfloat162_rn(x.v[2], x.v[3]);
    uint2 t;
    t.x = *reinterpret_cast<const unsigned*>(&a);
    t.y = *reinterpret_cast<const unsigned*>(&b);
    *reinterpret_cast<uint2*>(p) = t;
  } else {
    p[0] = __float2bfloat16_rn(x.v[0]);
  }
}

struct StepArgs {
  void* out;               // [R, W] or null (no norm)
  const float* x;          // [T, W]
  const void* y;           // [T, W] or null
  float mult;
  float* keep;             // [T, W] or null
  float* x_out;            // [T, W] or null
  const float* dw;         // [n + 2] or null
  const float* first;      // E [T, W]
  const float* later;      // P [n, T, W], later_stride values apart
  long long later_stride;
  int n;
  int norm;                // 0 none, 1 RMS, 2 layer norm
  const float* w;
  const float* b;          // or null
  float eps;
  const int* rows;
  int W;
};

template <typename TOut, typename TDelta, int VEC, int VPT>
__global__ void __launch_bounds__(DEPTH_THREADS)
residual_step_kernel(StepArgs a) {
  __shared__ float scratch[33];
  using V = Values<VEC>;
  const int r = blockIdx.x, W = a.W;
  const int row = a.rows ? a.rows[r] : r;                 // the row list is part of the step's description: no kernel writes it
  const size_t base = (size_t)row * W;
  mi::grid_dependency_sync();
  V cur[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int h = ((int)threadIdx.x + i * (int)blockDim.x) * VEC;
#pragma unroll
    for (int c = 0; c < VEC; ++c) cur[i].v[c] = 0.f;
    if (h >= W) continue;
    cur[i] = depth_load<VEC>(a.x + base + h);
    if (a.y) {
      const V d = depth_load<VEC>((const TDelta*)a.y + base + h);
#pragma unroll
      for (int c = 0; c < VEC; ++c) cur[i].v[c] = fmaf(a.mult, d.v[c], cur[i].v[c]);
    }
    if (a.keep) depth_store<VEC>(a.keep + base + h, cur[i]);
  }
  if (a.dw) {
    // E and the P in turn, four terms on their way at a time; then X itself
    const int terms = a.n + 1;
    V acc[VPT];
#pragma unroll
    for (int i = 0; i < VPT; ++i)
#pragma unroll
      for (int c = 0; c < VEC; ++c) acc[i].v[c] = 0.f;
    for (int k0 = 0; k0 < terms; k0 += 4) {
      V t[4][VPT];
      float wk[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int k = k0 + u;
        wk[u] = k < terms ? a.dw[k] : 0.f;
        const float* src = (k == 0 ? a.first : a.later + (size_t)(k - 1) * a.later_stride) + base;
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int h = ((int)threadIdx.x + i * (int)blockDim.x) * VEC;
          if (k < terms && h < W) t[u][i] = depth_load<VEC>(src + h);
        }
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        if (k0 + u >= terms) break;
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int h = ((int)threadIdx.x + i * (int)blockDim.x) * VEC;
          if (h < W) {
#pragma unroll
            for (int c = 0; c < VEC; ++c) acc[i].v[c] = fmaf(wk[u], t[u][i].v[c], acc[i].v[c]);
          }
        }
      }
    }
    const float last = a.dw[terms];
#pragma unroll
    for (int i = 0; i < VPT; ++i)
#pragma unroll
      for (int c = 0; c < VEC; ++c) cur[i].v[c] = fmaf(last, cur[i].v[c], acc[i].v[c]);      // past the row's end both are 0
  }
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int h = ((int)threadIdx.x + i * (int)blockDim.x) * VEC;
    if (h >= W) continue;
    if (a.x_out) depth_store<VEC>(a.x_out + base + h, cur[i]);
#pragma unroll
    for (int c = 0; c < VEC; ++c) s += cur[i].v[c];
  }
  if (a.norm == 0) return;
  const float mean = a.norm == 2 ? mi::block_sum(s, scratch) / (float)W : 0.f;
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int h = ((int)threadIdx.x + i * (int)blockDim.x) * VEC;
    if (h >= W) continue;
#pragma unroll
    for (int c = 0; c < VEC; ++c) {
      cur[i].v[c] -= mean;
      q = fmaf(cur[i].v[c], cur[i].v[c], q);
    }
  }
  const float rstd = 1.f / sqrtf(mi::block_sum(q, scratch) / (float)W + a.eps);
  TOut* o = (TOut*)a.out + (size_t)r * W;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int h = ((int)threadIdx.x + i * (int)blockDim.x) * VEC;
    if (h >= W) continue;
    const V w = depth_load<VEC>(a.w + h);
    V y;
#pragma unroll
    for (int c = 0; c < VEC; ++c) y.v[c] = cur[i].v[c] * rstd * w.v[c];
    if (a.b) {
      const V b = depth_load<VEC>(a.b + h);
#pragma unroll
      for (int c = 0; c < VEC; ++c) y.v[c] += b.v[c];
    }
    depth_store<VEC>(o + h, y);
  }
}

template <typename TOut, typename TDelta>
int step_rows(const StepArgs& a, int R, cudaStream_t stream) {
  const int W = a.W;
  const uintptr_t floats = (uintptr_t)a.x | (uintptr_t)a.keep | (uintptr_t)a.x_out | (uintptr_t)a.first | (uintptr_t)a.later |
                           (uintptr_t)a.w | (uintptr_t)a.b | (uintptr_t)(a.later_stride * 4);
  const bool vec = W % 4 == 0 && floats % 16 == 0 && ((uintptr_t)a.out % (4 * sizeof(TOut))) == 0 && ((uintptr_t)a.y % (4 * sizeof(TDelta))) == 0;
  const int units = vec ? W / 4 : W;
  // the number of threads is a function of the width alone: it fixes the order of the sums
  const int threads = units < DEPTH_THREADS ? (units + 31) / 32 * 32 : DEPTH_THREADS;
  const int vpt = (units + threads - 1) / threads;
#define MI_STEP(V, P) mi::launch(residual_step_kernel<TOut, TDelta, V, P>, dim3(R), dim3(threads), 0, stream, a)
  if (vec && vpt <= 1) MI_STEP(4, 1);
  else if (vec && vpt <= 2) MI_STEP(4, 2);
  else if (vec && vpt <= 4) MI_STEP(4, 4);
  else if (!vec && vpt <= 2) MI_STEP(1, 2);
  else if (!vec && vpt <= 16) MI_STEP(1, 16);
  else return mi_fail("residual_step: rows of %d values are more than the kernel keeps in registers (16384)", W);
#undef MI_STEP
  MI_LAUNCH_OK("residual_step");
  return 0;
}

}  // namespace

MI_API int mi_residual_step(void* out, int out_dtype, const float* x, const void* y, int y_dtype, float mult, float* keep, float* x_out,
                            const float* dw, const float* first, const float* later, long long later_stride, int n, int norm,
                            const float* w, const float* b, float eps, const int* rows, int R, int W, cudaStream_t stream) {
  MI_REQUIRE(R >= 0 && W > 0 && n >= 0, "residual_step: bad sizes R=%d W=%d n=%d", R, W, n);
  MI_REQUIRE(norm >= 0 && norm <= 2 && (norm == 0 || (out != nullptr && w != nullptr && eps > 0.f)), "residual_step: norm %d without its weight, eps or output", norm);
  MI_REQUIRE(dw == nullptr || (first != nullptr && (n == 0 || later != nullptr)), "residual_step: an average without its terms");
  if (R == 0) return 0;
  StepArgs a;
  a.out = out; a.x = x; a.y = y; a.mult = mult; a.keep = keep; a.x_out = x_out; a.dw = dw; a.first = first; a.later = later;
  a.later_stride = later_stride; a.n = n; a.norm = norm; a.w = w; a.b = b; a.eps = eps; a.rows = rows; a.W = W;
  if (out_dtype == MI_BF16 && y_dtype == MI_BF16) return step_rows<__nv_bfloat16, __nv_bfloat16>(a, R, stream);
  if (out_dtype == MI_F32 && y_dtype == MI_F32) return step_rows<float, float>(a, R, stream);
  return mi_fail("residual_step: unknown dtypes out=%d y=%d", out_dtype, y_dtype);
}
