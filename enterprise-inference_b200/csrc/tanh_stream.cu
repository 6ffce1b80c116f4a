// Parallel layer form with an elementwise norm (b200_stack_cfg.norm_kind = B200_NORM_TANH): what happens to the fp32 stream between
// two layers, and the inputs of its attention mixer.
//
//  * tanh_close: x += sa ya + sb yb + (sum of the experts' rows) + gate y_shared, then D(x) = tanh(alpha x) w + b for the layer that
//    follows.  D needs no statistics of the row, so the whole step is elementwise: CTAs take columns of a row, four neighbours per
//    thread, every input read once and every output written once.  Over the logit rows (row indirection) the stream is only read.
//  * qk_norm_cache: q and k brought to unit RMS over the WHOLE projection, times weights of that size; v as it is.  q leaves as fp32
//    rows, k and v go to the paged caches.  One CTA per row, the row staged in shared memory as fp32.
// All arithmetic fp32; sums in a fixed order, so a row's result does not depend on what else is in the step.
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

constexpr int kCloseThreads = 128;

template <typename AT>
struct CloseArgs {
  float* x;
  const AT *ya, *yb, *y_sh;
  const float *parts, *sh_gate, *alpha, *w, *b;
  AT* out;
  const int32_t* rows;
  float sa, sb;
  int n_parts, width;
};

template <typename AT, int V>
__global__ void __launch_bounds__(kCloseThreads)
tanh_close_kernel(const CloseArgs<AT> a) {
  const int c = (blockIdx.y * kCloseThreads + threadIdx.x) * V;
  if (c >= a.width) {
    pdl_wait();
    return;
  }
  // norm parameters are weights: they do not wait for the launch before
  float alpha = 0.f, w[V], b[V];
  if (a.out) {
    alpha = a.alpha[0];
    ldv<float, V>(a.w, c, w);
    ldv<float, V>(a.b, c, b);
  }
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = a.rows ? a.rows[blockIdx.x] : blockIdx.x, o = t * a.width + c;
  float x[V], y[V], s[V];
  ldv<float, V>(a.x, o, x);
#pragma unroll
  for (int v = 0; v < V; ++v) s[v] = 0.f;
  if (a.ya) {
    ldv<AT, V>(a.ya, o, y);
#pragma unroll
    for (int v = 0; v < V; ++v) s[v] = a.sa * y[v];
  }
  if (a.yb) {
    ldv<AT, V>(a.yb, o, y);
#pragma unroll
    for (int v = 0; v < V; ++v) s[v] = fmaf(a.sb, y[v], s[v]);
  }
  if (a.n_parts) {
    float f[V];
#pragma unroll
    for (int v = 0; v < V; ++v) f[v] = 0.f;
    const float* p = a.parts + t * a.n_parts * a.width + c;
#pragma unroll 4
    for (int k = 0; k < a.n_parts; ++k) {
      ldv<float, V>(p, (int64_t)k * a.width, y);
#pragma unroll
      for (int v = 0; v < V; ++v) f[v] += y[v];
    }
    if (a.y_sh) {
      ldv<AT, V>(a.y_sh, o, y);
      const float g = a.sh_gate ? a.sh_gate[t] : 1.0f;
#pragma unroll
      for (int v = 0; v < V; ++v) f[v] = fmaf(g, y[v], f[v]);
    }
#pragma unroll
    for (int v = 0; v < V; ++v) s[v] += f[v];
  }
#pragma unroll
  for (int v = 0; v < V; ++v) x[v] += s[v];
  if (a.ya && !a.rows) stv<float, V>(a.x, o, x);
  if (a.out) {
#pragma unroll
    for (int v = 0; v < V; ++v) y[v] = fmaf(tanhf(alpha * x[v]), w[v], b[v]);
    stv<AT, V>(a.out, (int64_t)blockIdx.x * a.width + c, y);
  }
}

template <typename AT>
int tanh_close_t(const CloseArgs<AT>& a, int R, cudaStream_t s) {
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.ya) | reinterpret_cast<uintptr_t>(a.yb) |
                         reinterpret_cast<uintptr_t>(a.y_sh) | reinterpret_cast<uintptr_t>(a.parts) | reinterpret_cast<uintptr_t>(a.w) |
                         reinterpret_cast<uintptr_t>(a.b) | reinterpret_cast<uintptr_t>(a.out);
  const bool v4 = a.width % 4 == 0 && ptrs % 16 == 0;
  const int per = kCloseThreads * (v4 ? 4 : 1);
  const dim3 grid(R, (a.width + per - 1) / per);
  if (v4) B200_CUDA(launch(tanh_close_kernel<AT, 4>, grid, dim3(kCloseThreads), (size_t)0, s, a));
  else B200_CUDA(launch(tanh_close_kernel<AT, 1>, grid, dim3(kCloseThreads), (size_t)0, s, a));
  return B200_OK;
}

// ---- attention inputs --------------------------------------------------------------------------------------------------------
constexpr int kQkThreads = 256;

__device__ __forceinline__ float block_sum_qk(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float r = 0.f;
#pragma unroll
  for (int i = 0; i < kQkThreads / 32; ++i) r += red[i];
  return r;
}

template <typename AT, int V>
__global__ void __launch_bounds__(kQkThreads)
qk_norm_cache_kernel(const AT* __restrict__ fused, int64_t ld, const float* __restrict__ qw, const float* __restrict__ kw,
                     const int32_t* __restrict__ slots, float* __restrict__ qout, AT* __restrict__ kc, AT* __restrict__ vc, int heads, int kv_heads,
                     int dim, int vdim, int block_size, float eps) {
  extern __shared__ __align__(16) float row[];   // [heads dim + kv_heads dim]
  __shared__ float red[kQkThreads / 32];
  const int64_t t = blockIdx.x;
  const int qn = heads * dim, kn = kv_heads * dim, vn = kv_heads * vdim;
  const int slot = slots[t];
  const int64_t blk = slot >= 0 ? slot / block_size : 0, off = slot >= 0 ? slot % block_size : 0;
  pdl_wait();
  pdl_launch_dependents();
  const AT* src = fused + t * ld;
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * V; c < qn + kn; c += kQkThreads * V) {
    float v[V];
    ldv<AT, V>(src, c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      row[c + i] = v[i];
      if (c < qn) sq = fmaf(v[i], v[i], sq);
      else sk = fmaf(v[i], v[i], sk);
    }
  }
  if (slot >= 0)
    for (int c = threadIdx.x * V; c < vn; c += kQkThreads * V) {
      float v[V];
      ldv<AT, V>(src, qn + kn + c, v);
      stv<AT, V>(vc, ((blk * kv_heads + c / vdim) * block_size + off) * vdim + c % vdim, v);
    }
  const float rq = 1.0f / sqrtf(block_sum_qk(sq, red) / (float)qn + eps);
  const float rk = 1.0f / sqrtf(block_sum_qk(sk, red) / (float)kn + eps);
  for (int c = threadIdx.x * V; c < qn + kn; c += kQkThreads * V) {   // a thread reads back what it staged itself
    const bool is_q = c < qn;
    const int e = is_q ? c : c - qn;
    float w[V], v[V];
    ldv<float, V>(is_q ? qw : kw, e, w);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = row[c + i] * (is_q ? rq : rk) * w[i];
    if (is_q) stv<float, V>(qout, t * qn + e, v);
    else if (slot >= 0) stv<AT, V>(kc, ((blk * kv_heads + e / dim) * block_size + off) * dim + e % dim, v);
  }
}

template <typename AT>
int qk_norm_cache_t(const void* fused, int64_t ld, const float* qw, const float* kw, const int32_t* slots, float* qout, void* kc, void* vc, int T,
                    int heads, int kv_heads, int dim, int vdim, int block_size, float eps, cudaStream_t s) {
  const size_t smem = (size_t)(heads + kv_heads) * dim * 4;
  B200_REQUIRE(smem <= 200 * 1024, B200_ERR_UNSUPPORTED, "qk_norm_cache: q|k rows of %zu bytes do not fit shared memory", smem);
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(fused) | reinterpret_cast<uintptr_t>(qw) | reinterpret_cast<uintptr_t>(kw) |
                         reinterpret_cast<uintptr_t>(qout) | reinterpret_cast<uintptr_t>(kc) | reinterpret_cast<uintptr_t>(vc);
  if (dim % 4 == 0 && vdim % 4 == 0 && ld % 4 == 0 && ptrs % 16 == 0) {
    static bool done[64] = {};
    if (smem > 48 * 1024) B200_CUDA(ensure_dynamic_smem(qk_norm_cache_kernel<AT, 4>, 200 * 1024, done));
    B200_CUDA(launch(qk_norm_cache_kernel<AT, 4>, dim3(T), dim3(kQkThreads), smem, s, (const AT*)fused, ld, qw, kw, slots, qout, (AT*)kc, (AT*)vc, heads,
                     kv_heads, dim, vdim, block_size, eps));
  } else {
    static bool done[64] = {};
    if (smem > 48 * 1024) B200_CUDA(ensure_dynamic_smem(qk_norm_cache_kernel<AT, 1>, 200 * 1024, done));
    B200_CUDA(launch(qk_norm_cache_kernel<AT, 1>, dim3(T), dim3(kQkThreads), smem, s, (const AT*)fused, ld, qw, kw, slots, qout, (AT*)kc, (AT*)vc, heads,
                     kv_heads, dim, vdim, block_size, eps));
  }
  return B200_OK;
}

}  // namespace

int tanh_close(bool f32, float* x, const void* ya, float sa, const void* yb, float sb, const float* parts, int n_parts, const void* y_sh,
               const float* sh_gate, const float* alpha, const float* w, const float* b, void* out, const int32_t* rows, int R, int width,
               cudaStream_t s) {
  if (R == 0) return B200_OK;
  B200_REQUIRE(!out || (alpha && w && b), B200_ERR_INVALID, "tanh_close: the norm needs alpha, weight and bias");
  B200_REQUIRE(ya || (!yb && !n_parts), B200_ERR_INVALID, "tanh_close: results without a first one");
  B200_REQUIRE(n_parts == 0 || parts, B200_ERR_INVALID, "tanh_close: no expert rows");
  B200_REQUIRE(!y_sh || n_parts, B200_ERR_INVALID, "tanh_close: a shared expert comes with routed ones");
  if (f32) {
    CloseArgs<float> a = {x, (const float*)ya, (const float*)yb, (const float*)y_sh, parts, sh_gate, alpha, w, b, (float*)out, rows, sa, sb, n_parts, width};
    return tanh_close_t<float>(a, R, s);
  }
  CloseArgs<__nv_bfloat16> a = {x, (const __nv_bfloat16*)ya, (const __nv_bfloat16*)yb, (const __nv_bfloat16*)y_sh, parts, sh_gate, alpha, w, b,
                                (__nv_bfloat16*)out, rows, sa, sb, n_parts, width};
  return tanh_close_t<__nv_bfloat16>(a, R, s);
}

int qk_norm_cache(bool f32, const void* fused, int64_t ld, const float* qw, const float* kw, const int32_t* slots, float* qout, void* kc, void* vc,
                  int T, int heads, int kv_heads, int dim, int vdim, int block_size, float eps, cudaStream_t s) {
  if (T == 0) return B200_OK;
  return f32 ? qk_norm_cache_t<float>(fused, ld, qw, kw, slots, qout, kc, vc, T, heads, kv_heads, dim, vdim, block_size, eps, s)
             : qk_norm_cache_t<__nv_bfloat16>(fused, ld, qw, kw, slots, qout, kc, vc, T, heads, kv_heads, dim, vdim, block_size, eps, s);
}

}  // namespace b200
