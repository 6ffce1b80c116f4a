// The row pass between two sublayers of the looped layer form (B200_FORM_LOOPED): an fp32 residual stream with RMS norms on both
// sides of every sublayer.  One launch closes a sublayer and opens the next:
//   v  = y                                          a sublayer's result, or
//   v  = (y_a r_a w_a + y_b r_b w_b) / 2            two mixers side by side, each brought to unit RMS (r = 1 / rms) times its weight
//   x += v / rms(v) * w_post;      x += e;   x += step       (e: the embedding output, step: a pass's vector; each optional)
//   out = x / rms(x) * w_next
// The first launch of a step (init) turns the gathered embedding rows into x = x / rms(x) * w_post and keeps them as e where a
// loop adds them again; the last one runs over the logit rows only and leaves the stream alone.
// One CTA per row; the row waits in shared memory between the statistics passes, all arithmetic is fp32.
#include <algorithm>

#include "common.cuh"

namespace b200 {
namespace {

template <typename AT, int V> __device__ __forceinline__ void ldv(const AT* p, int64_t i, float* o);
template <> __device__ __forceinline__ void ldv<float, 1>(const float* p, int64_t i, float* o) { o[0] = p[i]; }
template <> __device__ __forceinline__ void ldv<__nv_bfloat16, 1>(const __nv_bfloat16* p, int64_t i, float* o) { o[0] = __bfloat162float(p[i]); }
template <> __device__ __forceinline__ void ldv<float, 4>(const float* p, int64_t i, float* o) {
  const float4 v = *reinterpret_cast<const float4*>(p + i);
  o[0] = v.x, o[1] = v.y, o[2] = v.z, o[3] = v.w;
}
template <> __device__ __forceinline__ void ldv<__nv_bfloat16, 4>(const __nv_bfloat16* p, int64_t i, float* o) {
  const uint2 v = *reinterpret_cast<const uint2*>(p + i);
  o[0] = bf16lo(v.x), o[1] = bf16hi(v.x), o[2] = bf16lo(v.y), o[3] = bf16hi(v.y);
}
template <typename AT, int V> __device__ __forceinline__ void stv(AT* p, int64_t i, const float* o);
template <> __device__ __forceinline__ void stv<float, 1>(float* p, int64_t i, const float* o) { p[i] = o[0]; }
template <> __device__ __forceinline__ void stv<__nv_bfloat16, 1>(__nv_bfloat16* p, int64_t i, const float* o) { p[i] = __float2bfloat16_rn(o[0]); }
template <> __device__ __forceinline__ void stv<float, 4>(float* p, int64_t i, const float* o) {
  *reinterpret_cast<float4*>(p + i) = make_float4(o[0], o[1], o[2], o[3]);
}
template <> __device__ __forceinline__ void stv<__nv_bfloat16, 4>(__nv_bfloat16* p, int64_t i, const float* o) {
  *reinterpret_cast<uint2*>(p + i) = make_uint2(pack_bf16(o[0], o[1]), pack_bf16(o[2], o[3]));
}

// sums of two values over the CTA (any number of warps up to 32); red holds 64 floats
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
  a = warp_sum(a);
  b = warp_sum(b);
  const int nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) {
    red[threadIdx.x >> 5] = a;
    red[32 + (threadIdx.x >> 5)] = b;
  }
  __syncthreads();
  float sa = 0.f, sb = 0.f;
  for (int i = 0; i < nw; ++i) sa += red[i], sb += red[32 + i];
  return make_float2(sa, sb);
}
__device__ __forceinline__ float block_sum1(float a, float* red) { return block_sum2(a, 0.f, red).x; }

template <typename AT>
struct RmsArgs {
  float* x;
  const AT *y, *y_b;
  const float *w_a, *w_b, *w_post;
  int init;
  float *e_out, *tap;
  const float *e, *step, *w_next;
  AT* out;
  const int32_t* rows;
  int width;
  float eps;
};

template <typename AT, int V>
__global__ void __launch_bounds__(1024)
rms_sandwich_kernel(const RmsArgs<AT> a) {
  extern __shared__ __align__(16) float row[];
  __shared__ float red[64];
  const int width = a.width, nt = blockDim.x;
  if (gridDim.x <= 256) {   // short steps wait on latency: the weights go to L2 while the launch before runs
    if (a.w_a) prefetch_l2_span(a.w_a, (size_t)width * 4);
    if (a.w_b) prefetch_l2_span(a.w_b, (size_t)width * 4);
    if (a.w_post) prefetch_l2_span(a.w_post, (size_t)width * 4);
    if (a.w_next) prefetch_l2_span(a.w_next, (size_t)width * 4);
    if (a.step) prefetch_l2_span(a.step, (size_t)width * 4);
  }
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x, src = a.rows ? (int64_t)a.rows[t] : t, base = src * width;
  const float inv_w = 1.0f / (float)width;
  float ra = 0.f, rb = 0.f;
  if (a.y_b) {   // two results: their own statistics first
    float sa = 0.f, sb = 0.f;
    for (int c = threadIdx.x * V; c < width; c += nt * V) {
      float va[V], vb[V];
      ldv<AT, V>(a.y, base + c, va);
      ldv<AT, V>(a.y_b, base + c, vb);
#pragma unroll
      for (int v = 0; v < V; ++v) sa = fmaf(va[v], va[v], sa), sb = fmaf(vb[v], vb[v], sb);
    }
    const float2 s2 = block_sum2(sa, sb, red);
    ra = 0.5f / sqrtf(s2.x * inv_w + a.eps);
    rb = 0.5f / sqrtf(s2.y * inv_w + a.eps);
  }
  const bool close = a.y || a.init;
  float rv = 0.f;
  if (close) {
    float ss = 0.f;
    for (int c = threadIdx.x * V; c < width; c += nt * V) {
      float o[V];
      if (a.init) {
        ldv<float, V>(a.x, base + c, o);
      } else {
        ldv<AT, V>(a.y, base + c, o);
        if (a.y_b) {
          float vb[V], wa[V], wb[V];
          ldv<AT, V>(a.y_b, base + c, vb);
          ldv<float, V>(a.w_a, c, wa);
          ldv<float, V>(a.w_b, c, wb);
#pragma unroll
          for (int v = 0; v < V; ++v) o[v] = fmaf(vb[v] * rb, wb[v], o[v] * ra * wa[v]);
        }
      }
#pragma unroll
      for (int v = 0; v < V; ++v) ss = fmaf(o[v], o[v], ss);
      stv<float, V>(row, c, o);
    }
    rv = 1.0f / sqrtf(block_sum1(ss, red) * inv_w + a.eps);
  }
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < width; c += nt * V) {   // a thread meets the channels it staged
    float x[V];
    if (!a.init) ldv<float, V>(a.x, base + c, x);
    if (close) {
      float w[V], o[V];
      ldv<float, V>(a.w_post, c, w);
      ldv<float, V>(row, c, o);
#pragma unroll
      for (int v = 0; v < V; ++v) x[v] = a.init ? o[v] * rv * w[v] : fmaf(o[v] * rv, w[v], x[v]);
    }
    if (a.e_out) stv<float, V>(a.e_out, base + c, x);
    if (a.tap) stv<float, V>(a.tap, base + c, x);
    if (a.e) {
      float e[V];
      ldv<float, V>(a.e, base + c, e);
#pragma unroll
      for (int v = 0; v < V; ++v) x[v] += e[v];
    }
    if (a.step) {
      float st[V];
      ldv<float, V>(a.step, c, st);
#pragma unroll
      for (int v = 0; v < V; ++v) x[v] += st[v];
    }
    if (!a.rows && (close || a.e || a.step)) stv<float, V>(a.x, base + c, x);
    stv<float, V>(row, c, x);
#pragma unroll
    for (int v = 0; v < V; ++v) ss = fmaf(x[v], x[v], ss);
  }
  if (!a.w_next) return;
  const float rx = 1.0f / sqrtf(block_sum1(ss, red) * inv_w + a.eps);
  for (int c = threadIdx.x * V; c < width; c += nt * V) {
    float w[V], o[V];
    ldv<float, V>(a.w_next, c, w);
    ldv<float, V>(row, c, o);
#pragma unroll
    for (int v = 0; v < V; ++v) o[v] = o[v] * rx * w[v];
    stv<AT, V>(a.out, t * width + c, o);
  }
}

template <typename AT>
int rms_sandwich_t(const RmsArgs<AT>& a, int R, cudaStream_t s) {
  const size_t smem = (size_t)a.width * 4;
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.y_b) |
                         reinterpret_cast<uintptr_t>(a.w_a) | reinterpret_cast<uintptr_t>(a.w_b) | reinterpret_cast<uintptr_t>(a.w_post) |
                         reinterpret_cast<uintptr_t>(a.e_out) | reinterpret_cast<uintptr_t>(a.tap) | reinterpret_cast<uintptr_t>(a.e) |
                         reinterpret_cast<uintptr_t>(a.step) | reinterpret_cast<uintptr_t>(a.w_next) | reinterpret_cast<uintptr_t>(a.out);
  if (a.width % 4 == 0 && ptrs % 16 == 0) {
    // one trip per thread for short steps; long steps take small CTAs so that many share an SM and hide one another's block sums
    const int threads = R >= 512 ? 128 : std::min(1024, std::max(64, (a.width / 4 + 31) / 32 * 32));
    static bool done[64] = {};
    if (smem > 48 * 1024) B200_CUDA(ensure_dynamic_smem(rms_sandwich_kernel<AT, 4>, 200 * 1024, done));
    B200_CUDA(launch(rms_sandwich_kernel<AT, 4>, dim3(R), dim3(threads), smem, s, a));
    return B200_OK;
  }
  const int threads = std::min(1024, std::max(64, (a.width / 2 + 31) / 32 * 32));
  static bool done1[64] = {};
  if (smem > 48 * 1024) B200_CUDA(ensure_dynamic_smem(rms_sandwich_kernel<AT, 1>, 200 * 1024, done1));
  B200_CUDA(launch(rms_sandwich_kernel<AT, 1>, dim3(R), dim3(threads), smem, s, a));
  return B200_OK;
}

}  // namespace

int rms_sandwich(bool f32, float* x, const void* y, const void* y_b, const float* w_a, const float* w_b, const float* w_post, bool init,
                 float* e_out, float* tap, const float* e, const float* step, const float* w_next, void* out, const int32_t* rows, int R,
                 int width, float eps, cudaStream_t s) {
  if (R == 0) return B200_OK;
  B200_REQUIRE(!(y || init) || w_post, B200_ERR_INVALID, "rms_sandwich: a closing sublayer needs its norm weight");
  B200_REQUIRE(!(init && (y || rows)) && (!y_b || (y && w_a && w_b)) && (!w_next || out), B200_ERR_INVALID, "rms_sandwich: bad combination of arguments");
  B200_REQUIRE(!rows || (!e_out && !tap), B200_ERR_INVALID, "rms_sandwich: picked rows leave the stream alone");
  B200_REQUIRE((size_t)width * 4 <= 200 * 1024, B200_ERR_UNSUPPORTED, "rms_sandwich: width %d does not fit shared memory", width);
  if (f32) {
    RmsArgs<float> a = {x, (const float*)y, (const float*)y_b, w_a, w_b, w_post, init ? 1 : 0, e_out, tap, e, step, w_next, (float*)out, rows, width, eps};
    return rms_sandwich_t<float>(a, R, s);
  }
  RmsArgs<__nv_bfloat16> a = {x, (const __nv_bfloat16*)y, (const __nv_bfloat16*)y_b, w_a, w_b, w_post, init ? 1 : 0, e_out, tap, e, step, w_next,
                              (__nv_bfloat16*)out, rows, width, eps};
  return rms_sandwich_t<__nv_bfloat16>(a, R, s);
}

}  // namespace b200
