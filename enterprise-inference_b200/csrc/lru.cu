// Real-gated linear recurrent unit (B200_MIXER_LRU), per channel c of one sequence:
//   r = sigmoid(R u + br)_c,  i = sigmoid(I u + bi)_c              (R, I block-diagonal: head_linear gives the products in fp32)
//   a = exp(-r d_c),   S_t = a S_(t-1) + sqrt(1 - a^2) i u_t,   out_t = S_t gelu_tanh(y_t)
// u: convolved inputs, y: the other branch's projection, both of the activation type; gates, decays and S fp32.
//
//  * step kernel (every sequence brings one row): a thread per channel; the state is read ahead of the dependency wait.
//  * scan kernel: the recurrence is linear, so a run of rows acts on the state as S -> S - M S + B (M = 1 - the product of its decays).
//    A CTA takes 16 channels of one sequence and walks it in tiles of 32 segments x kLruRows rows: a thread folds its segment of one
//    channel (of two neighbouring ones where pairs are aligned) into (M, B), a warp joins the 32 pairs of a channel with shuffles and
//    hands every segment the state ahead of it, and the threads run their rows once more from there.  The next tile's inputs are
//    requested before the barriers of this one.
// A sequence whose first row of the step is at position 0 starts from zeros, whatever the slot held.
#include <algorithm>

#include "common.cuh"

namespace b200 {
namespace {

__device__ __forceinline__ float ldf(float v) { return v; }
__device__ __forceinline__ float ldf(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void stf(float* p, int64_t i, float v) { p[i] = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, int64_t i, float v) { p[i] = __float2bfloat16_rn(v); }

// One row of one channel, with z the decay gate's and g the input gate's logit: m = 1 - a and b = sqrt(1 - a^2) i u, 1 - a^2 = m (2 - m).
// The decays of a long memory are close to one; they are carried as m = 1 - e^-h, which keeps its relative precision there, and the
// state moves by S += b - m S: a decay that is off by a rounding would be off the same way at every row of the context.
// 32-bit mode: the library's functions.  Serving mode: the hardware's exponential, reciprocal and square root (fp32, a few units in the
// last place), and for small h the Taylor series of 1 - e^-h.
constexpr float kLog2e = 1.4426950408889634f;
__device__ __forceinline__ float hw_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float hw_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float hw_sqrt(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <typename AT>
__device__ __forceinline__ void lru_terms(float z, float g, float d, float u, float& m, float& b) {
  if constexpr (sizeof(AT) == 4) {
    const float r = 1.0f / (1.0f + expf(-z)), i = 1.0f / (1.0f + expf(-g));
    m = -expm1f(-r * d);
    b = sqrtf(m * (2.0f - m)) * i * u;
  } else {
    const float r = hw_rcp(1.0f + hw_exp2(-kLog2e * z)), i = hw_rcp(1.0f + hw_exp2(-kLog2e * g)), h = r * d;
    const float series = h * fmaf(h, fmaf(h, fmaf(h, fmaf(h, fmaf(h, -1.0f / 720.0f, 1.0f / 120.0f), -1.0f / 24.0f), 1.0f / 6.0f), -0.5f), 1.0f);
    m = h < 0.25f ? series : 1.0f - hw_exp2(-kLog2e * h);
    b = hw_sqrt(m * (2.0f - m)) * (i * u);
  }
}
__device__ __forceinline__ float lru_move(float S, float m, float b) { return S + fmaf(-m, S, b); }

// gelu_tanh(y); 0.5 (1 + tanh(w)) = 1 / (1 + e^-2w)
template <typename AT>
__device__ __forceinline__ float branch_gelu(float y) {
  if constexpr (sizeof(AT) == 4) return act_apply(y, B200_ACT_GELU_TANH);
  else return y * hw_rcp(1.0f + hw_exp2((-1.5957691216057308f * kLog2e) * fmaf(0.044715f * y * y, y, y)));
}

template <typename AT>
struct LruArgs {
  const AT* u;
  const float *gates, *gate_bias, *decay;
  const AT* y;
  int64_t ldy;
  const int32_t *positions, *seq_start, *seq_slots;
  float* state;
  int64_t slot_stride;
  AT* out;
  int width, block;
};

constexpr int kStepThreads = 128;
template <typename AT>
__global__ void __launch_bounds__(kStepThreads)
lru_step_kernel(const LruArgs<AT> p) {
  const int64_t t = blockIdx.x;
  const int c = blockIdx.y * kStepThreads + threadIdx.x;
  if (c >= p.width) {
    pdl_wait();
    return;
  }
  const int ir = 2 * (c / p.block) * p.block + c % p.block, ii = ir + p.block;   // this channel's rows among the gates
  float* st = p.state + (int64_t)p.seq_slots[t] * p.slot_stride + c;
  const float S0 = p.positions[t] == 0 ? 0.f : *st, d = p.decay[c], br = p.gate_bias[ir], bi = p.gate_bias[ii];
  pdl_wait();
  pdl_launch_dependents();
  const float* g = p.gates + t * 2 * p.width;
  float m, b;
  lru_terms<AT>(g[ir] + br, g[ii] + bi, d, ldf(p.u[t * p.width + c]), m, b);
  const float S = lru_move(S0, m, b);
  *st = S;
  stf(p.out, t * p.width + c, S * branch_gelu<AT>(ldf(p.y[t * p.ldy + c])));
}

constexpr int kLruCh = 16, kLruSegs = 32, kLruRows = 4;
// V neighbouring channels per thread (2: pairs of channels and rows are there in 8 bytes)
template <int V> __device__ __forceinline__ void ldc(const float* p, float* o) {
  if constexpr (V == 2) {
    const float2 v = *reinterpret_cast<const float2*>(p);
    o[0] = v.x, o[1] = v.y;
  } else {
    o[0] = *p;
  }
}
template <int V> __device__ __forceinline__ void ldc(const __nv_bfloat16* p, uint32_t* o) {
  if constexpr (V == 2) *o = *reinterpret_cast<const uint32_t*>(p);
  else *o = *reinterpret_cast<const unsigned short*>(p);
}
template <int V> __device__ __forceinline__ void widen(const float* r, float* o) {
#pragma unroll
  for (int v = 0; v < V; ++v) o[v] = r[v];
}
template <int V> __device__ __forceinline__ void widen(const uint32_t* r, float* o) {
  o[0] = bf16lo(*r);
  if constexpr (V == 2) o[1] = bf16hi(*r);
}
template <int V> __device__ __forceinline__ void stc(float* p, const float* o) {
  if constexpr (V == 2) *reinterpret_cast<float2*>(p) = make_float2(o[0], o[1]);
  else *p = o[0];
}
template <int V> __device__ __forceinline__ void stc(__nv_bfloat16* p, const float* o) {
  if constexpr (V == 2) *reinterpret_cast<uint32_t*>(p) = pack_bf16(o[0], o[1]);
  else *p = __float2bfloat16_rn(o[0]);
}
template <typename AT, int V> struct LruRaw { uint32_t r; };
template <int V> struct LruRaw<float, V> { float r[V]; };
__device__ __forceinline__ uint32_t* raw_of(LruRaw<__nv_bfloat16, 1>& v) { return &v.r; }
__device__ __forceinline__ uint32_t* raw_of(LruRaw<__nv_bfloat16, 2>& v) { return &v.r; }
template <int V> __device__ __forceinline__ float* raw_of(LruRaw<float, V>& v) { return v.r; }

template <typename AT, int V>
__global__ void __launch_bounds__(kLruCh / V * kLruSegs, V == 2 ? 2 : 1)
lru_scan_kernel(const LruArgs<AT> p) {
  constexpr int kPer = kLruCh / V;              // threads per segment
  __shared__ float2 ab[kLruCh][kLruSegs + 1];
  __shared__ float sin_[kLruCh][kLruSegs + 1];
  const int s = blockIdx.x, ch = threadIdx.x % kPer * V, seg = threadIdx.x / kPer, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.y * kLruCh + ch, cc = min(c, p.width - V);   // V == 2: the width is even
  const bool live = c < p.width;
  const int start = p.seq_start[s], n_rows = p.seq_start[s + 1] - start;
  if (n_rows <= 0) {
    pdl_wait();
    return;
  }
  const int ir = 2 * (cc / p.block) * p.block + cc % p.block, ii = ir + p.block;
  float d[V], br[V], bi[V];
  ldc<V>(p.decay + cc, d);
  ldc<V>(p.gate_bias + ir, br);
  ldc<V>(p.gate_bias + ii, bi);
  // warp w carries the channels w V .. w V + V - 1 of the CTA from tile to tile
  float carry[V];
  float* st = p.state + (int64_t)p.seq_slots[s] * p.slot_stride;
  const bool fresh = p.positions[start] == 0;
#pragma unroll
  for (int v = 0; v < V; ++v) carry[v] = fresh ? 0.f : st[min((int)blockIdx.y * kLruCh + warp * V + v, p.width - 1)];
  pdl_wait();
  pdl_launch_dependents();
  constexpr int kTile = kLruSegs * kLruRows;
  float zr[kLruRows][V], zi[kLruRows][V];
  LruRaw<AT, V> ur[kLruRows], yr[kLruRows];
  const float* gp = p.gates + (int64_t)start * 2 * p.width;
  const AT *up = p.u + (int64_t)start * p.width + cc, *yp = p.y + (int64_t)start * p.ldy + cc;
  auto fetch = [&](int b0) {   // rows past the end are read at the last one and dropped below
#pragma unroll
    for (int k = 0; k < kLruRows; ++k) {
      const int64_t t = min(b0 + seg * kLruRows + k, n_rows - 1);
      const float* g = gp + t * 2 * p.width;
      ldc<V>(g + ir, zr[k]);
      ldc<V>(g + ii, zi[k]);
      ldc<V>(up + t * p.width, raw_of(ur[k]));
      ldc<V>(yp + t * p.ldy, raw_of(yr[k]));
    }
  };
  fetch(0);
  for (int b0 = 0; b0 < n_rows; b0 += kTile) {
    float m[kLruRows][V], b[kLruRows][V], y[kLruRows][V], M[V], B[V];   // the segment: S -> S - M S + B
    const int r0 = b0 + seg * kLruRows;
#pragma unroll
    for (int v = 0; v < V; ++v) M[v] = B[v] = 0.f;
#pragma unroll
    for (int k = 0; k < kLruRows; ++k) {
      float u[V];
      widen<V>(raw_of(ur[k]), u);
      widen<V>(raw_of(yr[k]), y[k]);
      const bool past = r0 + k >= n_rows;
#pragma unroll
      for (int v = 0; v < V; ++v) {
        lru_terms<AT>(zr[k][v] + br[v], zi[k][v] + bi[v], d[v], u[v], m[k][v], b[k][v]);
        if (past) m[k][v] = b[k][v] = 0.f;
        M[v] = lru_move(M[v], m[k][v], m[k][v]);
        B[v] = lru_move(B[v], m[k][v], b[k][v]);
      }
    }
    if (b0 + kTile < n_rows) fetch(b0 + kTile);   // travels while the segments are joined and the rows run again
#pragma unroll
    for (int v = 0; v < V; ++v) ab[ch + v][seg] = make_float2(M[v], B[v]);
    __syncthreads();
#pragma unroll
    for (int v = 0; v < V; ++v) {
      float2 f = ab[warp * V + v][lane];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {   // inclusive: the map of segments 0 .. lane
        const float pa = __shfl_up_sync(0xffffffffu, f.x, o), pb = __shfl_up_sync(0xffffffffu, f.y, o);
        if (lane >= o) {
          f.y = lru_move(pb, f.x, f.y);
          f.x = lru_move(pa, f.x, f.x);
        }
      }
      const float after = lru_move(carry[v], f.x, f.y), before = __shfl_up_sync(0xffffffffu, after, 1);
      sin_[warp * V + v][lane] = lane == 0 ? carry[v] : before;
      carry[v] = __shfl_sync(0xffffffffu, after, 31);
    }
    __syncthreads();
    float S[V];
#pragma unroll
    for (int v = 0; v < V; ++v) S[v] = sin_[ch + v][seg];
    AT* op = p.out + (int64_t)(start + r0) * p.width + c;
#pragma unroll
    for (int k = 0; k < kLruRows; ++k) {
      float o[V];
#pragma unroll
      for (int v = 0; v < V; ++v) {
        S[v] = lru_move(S[v], m[k][v], b[k][v]);
        o[v] = S[v] * branch_gelu<AT>(y[k][v]);
      }
      if (live && r0 + k < n_rows) stc<V>(op + (int64_t)k * p.width, o);
    }
  }
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int wc = blockIdx.y * kLruCh + warp * V + v;
    if (lane == 0 && wc < p.width) st[wc] = carry[v];
  }
}

template <typename AT>
int gated_lru_t(const LruArgs<AT>& a, int S, bool one_row, cudaStream_t s) {
  if (one_row) B200_CUDA(launch(lru_step_kernel<AT>, dim3(S, (a.width + kStepThreads - 1) / kStepThreads), dim3(kStepThreads), (size_t)0, s, a));
  else {
    const uintptr_t ptrs = reinterpret_cast<uintptr_t>(a.u) | reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.gates) |
                           reinterpret_cast<uintptr_t>(a.gate_bias) | reinterpret_cast<uintptr_t>(a.decay) | reinterpret_cast<uintptr_t>(a.out);
    const dim3 grid(S, (a.width + kLruCh - 1) / kLruCh);
    if (a.width % 2 == 0 && a.block % 2 == 0 && a.ldy % 2 == 0 && ptrs % (2 * sizeof(AT)) == 0 && ptrs % 4 == 0 &&
        (reinterpret_cast<uintptr_t>(a.gates) | reinterpret_cast<uintptr_t>(a.gate_bias) | reinterpret_cast<uintptr_t>(a.decay)) % 8 == 0)
      B200_CUDA(launch(lru_scan_kernel<AT, 2>, grid, dim3(kLruCh / 2 * kLruSegs), (size_t)0, s, a));
    else
      B200_CUDA(launch(lru_scan_kernel<AT, 1>, grid, dim3(kLruCh * kLruSegs), (size_t)0, s, a));
  }
  return B200_OK;
}

}  // namespace

int gated_lru(bool f32, const void* u, const float* gates, const float* gate_bias, const float* decay, const void* y, int64_t ldy,
              const int32_t* positions, const int32_t* seq_start, const int32_t* seq_slots, float* state, int64_t slot_stride, void* out, int S,
              int width, int blocks, bool one_row, cudaStream_t s) {
  if (S == 0) return B200_OK;
  B200_REQUIRE(width > 0 && blocks > 0 && width % blocks == 0, B200_ERR_INVALID, "gated_lru: %d channels in %d parts", width, blocks);
  if (f32) {
    LruArgs<float> a = {(const float*)u, gates, gate_bias, decay, (const float*)y, ldy, positions, seq_start, seq_slots, state, slot_stride, (float*)out,
                        width, width / blocks};
    return gated_lru_t<float>(a, S, one_row, s);
  }
  LruArgs<__nv_bfloat16> a = {(const __nv_bfloat16*)u, gates, gate_bias, decay, (const __nv_bfloat16*)y, ldy, positions, seq_start, seq_slots, state,
                              slot_stride, (__nv_bfloat16*)out, width, width / blocks};
  return gated_lru_t<__nv_bfloat16>(a, S, one_row, s);
}

}  // namespace b200
