// Inputs of an attention mixer whose q, k and v pass a short convolution, with a selective scan beside it (B200_MIXER_SELECTIVE), and
// the scan itself.
//
//  * conv_inputs: causal per-channel convolutions over the fused projection rows q | k | v | x.  A thread owns V channels and walks a
//    run of rows with the earlier inputs in registers, so every input is fetched once; ahead of a portion's first row they come from
//    the sequence's tails in its state slot.  q, k, v: no activation; q leaves as fp32 rows, k and v go to the paged caches.
//    x: bias and silu (or no activation), rows of the activation type (they are also the input of the scan's projection).  In a step whose
//    sequences bring one row each (decode) the thread that read a channel's tail also shifts it.
//  * selective_scan: per channel c and state n   S = exp(dt_c A[c][n]) S + dt_c x_c B_n;   y_c = sum_n S[c][n] C_n + D_c x_c;
//    out_c = y_c silu(z_c), dt = softplus(dt_pre + bias).  Channels and states do not interact except through the sum over n, so a
//    channel is walked by L neighbouring lanes with NS states each in registers; a CTA of 128 threads takes 128 / L channels of one
//    sequence and stages 16 or 32 rows at a time in shared memory, the next ones travelling into registers meanwhile.  Only one multiply-add per state is on
//    the chain from a row to the next; the exponentials depend on dt alone.  The state, fp32 [inner][n_state] in the sequence's slot,
//    is read ahead of the dependency wait: no launch of the same step before this one writes it.
//    A sequence whose first row of the step is at position 0 starts from zeros, whatever the slot held.
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

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }

constexpr int kConvThreads = 128;

template <typename AT>
struct ConvArgs {
  const AT* fused;
  int64_t ld;
  const float *conv_a, *conv_x, *bias_x;
  float *tails_a, *tails_x;
  int taps_a, taps_x;
  int64_t slot_stride;
  const int32_t *positions, *row_to_seq, *seq_start, *seq_slots, *slots;
  float* qout;
  AT *kc, *vc, *xc;
  int T, heads, kv_heads, dim, vdim, inner, block_size, one_row, run, blocks_a, silu_x;
};

// TAPS > 0: known at compile time, earlier inputs in registers; 0: any count, earlier inputs re-read
template <typename AT, int V, int TAPS>
__device__ __forceinline__ void conv_walk(const ConvArgs<AT>& a, bool is_x, int c, int col, int n_ch, const float* w, int taps_rt, float* tails) {
  const int taps = TAPS > 0 ? TAPS : taps_rt;
  float wr[TAPS > 0 ? TAPS : 1][V], bias[V];
  float h1[V], h2[V], h3[V];   // TAPS > 0: the inputs of lag 1, 2, 3
#pragma unroll
  for (int v = 0; v < V; ++v) h1[v] = h2[v] = h3[v] = bias[v] = 0.f;
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int v = 0; v < V; ++v) wr[j][v] = w ? w[(int64_t)(c + v) * taps + j] : 1.0f;
  }
  if (is_x && a.bias_x) ldv<float, V>(a.bias_x, c, bias);
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim;
  const int t0 = blockIdx.x * a.run, t1 = min(a.T, t0 + a.run);
  int last_seq = -1;
  for (int t = t0; t < t1; ++t) {
    const int s = a.row_to_seq ? a.row_to_seq[t] : t;
    const int r = t - a.seq_start[s], pos = a.positions[t];
    float* tail = tails ? tails + (int64_t)a.seq_slots[s] * a.slot_stride : nullptr;   // [taps - 1][n_ch]
    auto lagged = [&](int j, float* o) {   // the input of position pos - j, j >= 1
      if (pos - j < 0) {
#pragma unroll
        for (int v = 0; v < V; ++v) o[v] = 0.f;
      } else if (r - j >= 0) {
        ldv<AT, V>(a.fused, (int64_t)(t - j) * a.ld + col, o);
      } else {
        ldv<float, V>(tail, (int64_t)(taps - 1 + r - j) * n_ch + c, o);
      }
    };
    float cur[V], acc[V];
    ldv<AT, V>(a.fused, (int64_t)t * a.ld + col, cur);
    if constexpr (TAPS > 0) {
      if (s != last_seq) {
        if constexpr (TAPS > 1) lagged(1, h1);
        if constexpr (TAPS > 2) lagged(2, h2);
        if constexpr (TAPS > 3) lagged(3, h3);
        last_seq = s;
      }
#pragma unroll
      for (int v = 0; v < V; ++v) {
        float x = bias[v];
        if constexpr (TAPS > 3) x = fmaf(wr[TAPS - 4][v], h3[v], x);
        if constexpr (TAPS > 2) x = fmaf(wr[TAPS - 3][v], h2[v], x);
        if constexpr (TAPS > 1) x = fmaf(wr[TAPS - 2][v], h1[v], x);
        acc[v] = fmaf(wr[TAPS - 1][v], cur[v], x);
      }
      if (a.one_row) {   // entry i of the tail takes lag taps - 2 - i
        if constexpr (TAPS > 3) stv<float, V>(tail, (int64_t)(TAPS - 4) * n_ch + c, h2);
        if constexpr (TAPS > 2) stv<float, V>(tail, (int64_t)(TAPS - 3) * n_ch + c, h1);
        if constexpr (TAPS > 1) stv<float, V>(tail, (int64_t)(TAPS - 2) * n_ch + c, cur);
      }
#pragma unroll
      for (int v = 0; v < V; ++v) {
        h3[v] = h2[v];
        h2[v] = h1[v];
        h1[v] = cur[v];
      }
    } else {
#pragma unroll
      for (int v = 0; v < V; ++v) acc[v] = fmaf(w[(int64_t)(c + v) * taps + taps - 1], cur[v], bias[v]);
      for (int j = 1; j < taps; ++j) {
        float o[V];
        lagged(j, o);
#pragma unroll
        for (int v = 0; v < V; ++v) acc[v] = fmaf(w[(int64_t)(c + v) * taps + taps - 1 - j], o[v], acc[v]);
      }
      if (a.one_row) {   // entry i takes the input of lag taps - 2 - i: what it reads lies above all it has written
        for (int i = 0; i < taps - 1; ++i) {
          float o[V];
          if (i == taps - 2) {
#pragma unroll
            for (int v = 0; v < V; ++v) o[v] = cur[v];
          } else {
            lagged(taps - 2 - i, o);
          }
          stv<float, V>(tail, (int64_t)i * n_ch + c, o);
        }
      }
    }
    if (is_x) {
      if (a.silu_x) {
#pragma unroll
        for (int v = 0; v < V; ++v) acc[v] = silu_f(acc[v]);
      }
      stv<AT, V>(a.xc, (int64_t)t * a.inner + c, acc);
    } else if (c < nq) {
      stv<float, V>(a.qout, (int64_t)t * nq + c, acc);
    } else {
      const int slot = a.slots[t];
      if (slot < 0) continue;
      const int64_t blk = slot / a.block_size, off = slot % a.block_size;
      const bool is_k = c < nq + nk;
      const int e = is_k ? c - nq : c - nq - nk, d = is_k ? a.dim : a.vdim, g = e / d;
      stv<AT, V>(is_k ? a.kc : a.vc, ((blk * a.kv_heads + g) * a.block_size + off) * d + e % d, acc);
    }
  }
}

template <typename AT, int V>
__global__ void __launch_bounds__(kConvThreads)
conv_inputs_kernel(const ConvArgs<AT> a) {
  pdl_wait();
  pdl_launch_dependents();
  const int n_a = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim);
  const bool is_x = (int)blockIdx.y >= a.blocks_a;
  const int n_ch = is_x ? a.inner : n_a, by = is_x ? blockIdx.y - a.blocks_a : blockIdx.y;
  const int c = (by * kConvThreads + threadIdx.x) * V;
  if (c >= n_ch) return;
  const int col = is_x ? n_a + c : c;
  const float* w = is_x ? a.conv_x : a.conv_a;
  float* tails = is_x ? a.tails_x : a.tails_a;
  const int taps = is_x ? a.taps_x : a.taps_a;
  switch (taps) {
    case 0: case 1: conv_walk<AT, V, 1>(a, is_x, c, col, n_ch, w, 1, tails); break;
    case 2: conv_walk<AT, V, 2>(a, is_x, c, col, n_ch, w, 2, tails); break;
    case 3: conv_walk<AT, V, 3>(a, is_x, c, col, n_ch, w, 3, tails); break;
    case 4: conv_walk<AT, V, 4>(a, is_x, c, col, n_ch, w, 4, tails); break;
    default: conv_walk<AT, V, 0>(a, is_x, c, col, n_ch, w, taps, tails); break;
  }
}

template <typename AT>
int conv_inputs_t(ConvArgs<AT> a, cudaStream_t s) {
  a.run = a.one_row ? 1 : (a.T >= 1024 ? 16 : (a.T >= 128 ? 8 : 2));
  const int n_a = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim);
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(a.fused) | reinterpret_cast<uintptr_t>(a.tails_a) | reinterpret_cast<uintptr_t>(a.tails_x) |
                         reinterpret_cast<uintptr_t>(a.bias_x) | reinterpret_cast<uintptr_t>(a.qout) | reinterpret_cast<uintptr_t>(a.kc) |
                         reinterpret_cast<uintptr_t>(a.vc) | reinterpret_cast<uintptr_t>(a.xc);
  // four channels per thread: every group of channels and every row starts at a multiple of four elements
  const bool v4 = ptrs % 16 == 0 && a.ld % 4 == 0 && a.slot_stride % 4 == 0 && (n_a == 0 || (a.dim % 4 == 0 && a.vdim % 4 == 0)) && a.inner % 4 == 0;
  const int per = kConvThreads * (v4 ? 4 : 1);
  a.blocks_a = (n_a + per - 1) / per;
  const int blocks_x = (a.inner + per - 1) / per;
  const dim3 grid((a.T + a.run - 1) / a.run, a.blocks_a + blocks_x);
  if (v4) B200_CUDA(launch(conv_inputs_kernel<AT, 4>, grid, dim3(kConvThreads), (size_t)0, s, a));
  else B200_CUDA(launch(conv_inputs_kernel<AT, 1>, grid, dim3(kConvThreads), (size_t)0, s, a));
  return B200_OK;
}

// ---- the scan ----------------------------------------------------------------------------------------------------------------
constexpr int kSelThreads = 128;

__device__ __forceinline__ float ldf(float v) { return v; }
__device__ __forceinline__ float ldf(__nv_bfloat16 v) { return __bfloat162float(v); }

// exp(x log 2) of the decays: the 32-bit mode takes the library's exp2f, the serving mode the hardware's approximation of it (two
// units in the last place, in fp32 as well)
template <typename AT> __device__ __forceinline__ float decay_exp2(float x);
template <> __device__ __forceinline__ float decay_exp2<float>(float x) { return exp2f(x); }
template <> __device__ __forceinline__ float decay_exp2<__nv_bfloat16>(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// four rows' partial sums over L neighbouring lanes -> the row totals; lane l of a group holds row l & 3 (L >= 4) or all four (L < 4)
template <int L>
__device__ __forceinline__ void group_sums(float (&y)[4], int lane) {
  if constexpr (L >= 4) {   // transposing: three exchanges for four sums, then plain rounds over the groups of four
    const bool o1 = lane & 1, o2 = lane & 2;
    const float a = __shfl_xor_sync(0xffffffffu, o1 ? y[0] : y[1], 1), b = __shfl_xor_sync(0xffffffffu, o1 ? y[2] : y[3], 1);
    const float p = (o1 ? y[1] : y[0]) + a, q = (o1 ? y[3] : y[2]) + b;   // rows (lane & 1) and 2 + (lane & 1)
    float r = (o2 ? q : p) + __shfl_xor_sync(0xffffffffu, o2 ? p : q, 2);
#pragma unroll
    for (int o = 4; o < L; o <<= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
    y[0] = r;
  } else {
#pragma unroll
    for (int o = 1; o < L; o <<= 1)
#pragma unroll
      for (int i = 0; i < 4; ++i) y[i] += __shfl_xor_sync(0xffffffffu, y[i], o);
  }
}

template <typename AT>
struct SelArgs {
  const AT *xc, *bc, *z;
  int64_t ldbc, ldz, slot_stride;
  int b_off;
  const float *dt_pre, *dt_bias, *A, *D;
  const int32_t *positions, *seq_start, *seq_slots;
  float* state;
  AT* out;
  int inner, n_state;
};

template <typename AT, int L, int NS>
__global__ void __launch_bounds__(kSelThreads)
selective_scan_kernel(const SelArgs<AT> a) {
  constexpr int kSelStage = L >= 2 && L * NS <= 32 ? 32 : 16;                                            // rows staged at a time
  constexpr int CH = kSelThreads / L, NP = L * NS;                                       // channels of the CTA, padded states
  constexpr int EX = (kSelStage * CH + kSelThreads - 1) / kSelThreads;                    // staged elements per thread: channel rows ..
  constexpr int EB = (kSelStage * NP + kSelThreads - 1) / kSelThreads;                    // .. B and C rows
  __shared__ __align__(16) float sB[kSelStage][NP], sC[kSelStage][NP];
  __shared__ float2 sd[kSelStage][CH];   // dt, dt x
  __shared__ float sy[kSelStage][CH];
  const int s = blockIdx.x, c0 = blockIdx.y * CH, tid = threadIdx.x;
  const int ch = tid / L, n0 = (tid % L) * NS, c = c0 + ch;
  const int N = a.n_state, inner = a.inner;
  float A[NS], S[NS];
  // bounds of the sequence, slots and positions are inputs of the step, the state is the step before's: all are complete when this
  // launch may start, so they are fetched while the launch before still runs
  const int start = a.seq_start[s], n_rows = a.seq_start[s + 1] - start;
  if (n_rows <= 0) {
    pdl_wait();
    return;
  }
  const bool fresh = a.positions[start] == 0;
  float* st = a.state + (int64_t)a.seq_slots[s] * a.slot_stride + (int64_t)c * N;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const bool live = c < inner && n0 + i < N;
    A[i] = live ? a.A[(int64_t)c * N + n0 + i] * 1.4426950408889634f : 0.f;   // log2(e): decays are powers of two
    S[i] = live && !fresh ? st[n0 + i] : 0.f;
  }
  pdl_wait();
  pdl_launch_dependents();
  // A thread stages one channel of rows r0, r0 + L, ...  What is not there is read at a clamped address and dropped when it is
  // staged: no branch and no conversion stands between the loads, so that all of them are in flight together.
  const int xc_ch = tid % CH, r0 = tid / CH, ccx = min(c0 + xc_ch, inner - 1);
  const bool live_x = c0 + xc_ch < inner;
  const float dtb = a.dt_bias[ccx], skip = a.D[ccx];
  AT rx[EX], rz[EX], rB[EB], rC[EB];
  float rdt[EX];
  auto fetch = [&](int b0) {
    const int last = min(kSelStage, n_rows - b0) - 1;
    const int64_t row = start + b0;
#pragma unroll
    for (int i = 0; i < EX; ++i) {
      const int64_t t = row + min(r0 + L * i, last);
      rx[i] = a.xc[t * inner + ccx];
      rdt[i] = a.dt_pre[t * inner + ccx];
      rz[i] = a.z[t * a.ldz + ccx];
    }
#pragma unroll
    for (int i = 0; i < EB; ++i) {
      const int e = tid + kSelThreads * i;
      const AT* p = a.bc + (row + min(e / NP, last)) * a.ldbc + a.b_off + min(e % NP, N - 1);
      rB[i] = p[0];
      rC[i] = p[N];
    }
  };
  fetch(0);
  for (int b0 = 0; b0 < n_rows; b0 += kSelStage) {
    const int nb = min(kSelStage, n_rows - b0);
    float xk[EX];   // this stage's x and gates, for the outputs
    AT zk[EX];
#pragma unroll
    for (int i = 0; i < EX; ++i) {
      const int r = r0 + L * i;
      const float x = ldf(rx[i]);
      xk[i] = x;
      zk[i] = rz[i];
      if (EX * kSelThreads == kSelStage * CH || r < kSelStage) {
        const float dt = r < nb && live_x ? softplus_f(rdt[i] + dtb) : 0.f;
        sd[r][xc_ch] = make_float2(dt, dt * x);
      }
    }
#pragma unroll
    for (int i = 0; i < EB; ++i) {
      const int e = tid + kSelThreads * i;
      if (EB * kSelThreads == kSelStage * NP || e < kSelStage * NP) {
        const bool live = e / NP < nb && e % NP < N;
        sB[e / NP][e % NP] = live ? ldf(rB[i]) : 0.f;
        sC[e / NP][e % NP] = live ? ldf(rC[i]) : 0.f;
      }
    }
    __syncthreads();
    if (b0 + kSelStage < n_rows) fetch(b0 + kSelStage);
    // four rows at a time: everything but the state's own chain is independent of the rows before (rows past nb have dt = 0 and
    // leave the state as it is)
    for (int r = 0; r < nb; r += 4) {
      float2 d[4];
      float dec[4][NS], u[4][NS], y[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) d[k] = sd[r + k][ch];
#pragma unroll
      for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int i = 0; i < NS; i += 4) {
          const float4 b = *reinterpret_cast<const float4*>(&sB[r + k][n0 + i]);
          u[k][i] = d[k].y * b.x, u[k][i + 1] = d[k].y * b.y, u[k][i + 2] = d[k].y * b.z, u[k][i + 3] = d[k].y * b.w;
#pragma unroll
          for (int x = 0; x < 4; ++x) dec[k][i + x] = decay_exp2<AT>(d[k].x * A[i + x]);
        }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        y[k] = 0.f;
#pragma unroll
        for (int i = 0; i < NS; i += 4) {
          const float4 q = *reinterpret_cast<const float4*>(&sC[r + k][n0 + i]);
          S[i] = fmaf(dec[k][i], S[i], u[k][i]), S[i + 1] = fmaf(dec[k][i + 1], S[i + 1], u[k][i + 1]);
          S[i + 2] = fmaf(dec[k][i + 2], S[i + 2], u[k][i + 2]), S[i + 3] = fmaf(dec[k][i + 3], S[i + 3], u[k][i + 3]);
          y[k] = fmaf(S[i], q.x, y[k]), y[k] = fmaf(S[i + 1], q.y, y[k]), y[k] = fmaf(S[i + 2], q.z, y[k]), y[k] = fmaf(S[i + 3], q.w, y[k]);
        }
      }
      group_sums<L>(y, tid);
      if constexpr (L >= 4) {
        if (tid % L < 4) sy[r + tid % L][ch] = y[0];
      } else {
        if (tid % L == 0) {
#pragma unroll
          for (int k = 0; k < 4; ++k) sy[r + k][ch] = y[k];
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < EX; ++i) {
      const int r = r0 + L * i;
      if (r < nb && live_x) {
        float o1[1] = {fmaf(skip, xk[i], sy[r][xc_ch]) * silu_f(ldf(zk[i]))};
        stv<AT, 1>(a.out, (int64_t)(start + b0 + r) * inner + ccx, o1);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NS; ++i)
    if (c < inner && n0 + i < N) st[n0 + i] = S[i];
}

// Every sequence of the step brings one row (decode): sequence s is row s.  No staging and no barrier: a thread takes KB groups of
// channels, 128 / L apart, with all their states and inputs in flight at once.
template <typename AT, int L, int NS, int KB>
__global__ void __launch_bounds__(kSelThreads)
selective_step_kernel(const SelArgs<AT> a, int vec) {
  constexpr int CH = kSelThreads / L;
  const int64_t t = blockIdx.x;
  const int c0 = blockIdx.y * CH * KB + threadIdx.x / L, n0 = (threadIdx.x % L) * NS, N = a.n_state, inner = a.inner;
  const bool fresh = a.positions[t] == 0;
  float* st = a.state + (int64_t)a.seq_slots[t] * a.slot_stride;
  float A[KB][NS], S[KB][NS];
#pragma unroll
  for (int k = 0; k < KB; ++k) {
    const int c = min(c0 + k * CH, inner - 1);
    if (vec) {   // N a multiple of 4, rows 16-byte aligned: a lane's states are there in fours
#pragma unroll
      for (int i = 0; i < NS; i += 4) {
        const int64_t o = (int64_t)c * N + min(n0 + i, N - 4);
        ldv<float, 4>(a.A, o, &A[k][i]);
        ldv<float, 4>(st, o, &S[k][i]);
      }
    } else {
#pragma unroll
      for (int i = 0; i < NS; ++i) {
        const int64_t o = (int64_t)c * N + min(n0 + i, N - 1);
        A[k][i] = a.A[o];
        S[k][i] = st[o];
      }
    }
  }
  pdl_wait();
  pdl_launch_dependents();
  AT x[KB], z[KB];
  float dt[KB], dtb[KB], skip[KB], B[NS], C[NS];
#pragma unroll
  for (int k = 0; k < KB; ++k) {
    const int c = min(c0 + k * CH, inner - 1);
    x[k] = a.xc[t * inner + c];
    dt[k] = a.dt_pre[t * inner + c];
    z[k] = a.z[t * a.ldz + c];
    dtb[k] = a.dt_bias[c];
    skip[k] = a.D[c];
  }
  {
    AT b[NS], q[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const AT* p = a.bc + t * a.ldbc + a.b_off + min(n0 + i, N - 1);
      b[i] = p[0];
      q[i] = p[N];
    }
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      B[i] = n0 + i < N ? ldf(b[i]) : 0.f;   // states past N stay out of the sums and are not stored
      C[i] = n0 + i < N ? ldf(q[i]) : 0.f;
    }
  }
#pragma unroll
  for (int k = 0; k < KB; ++k) {
    const int c = c0 + k * CH;
    const float d = softplus_f(dt[k] + dtb[k]), xv = ldf(x[k]), dx = d * xv;
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const float s0 = fresh ? 0.f : S[k][i];
      S[k][i] = fmaf(decay_exp2<AT>(d * (A[k][i] * 1.4426950408889634f)), s0, dx * B[i]);
      y = fmaf(S[k][i], C[i], y);
    }
#pragma unroll
    for (int o = 1; o < L; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (c < inner) {
      if (threadIdx.x % L == 0) {
        float o1[1] = {fmaf(skip[k], xv, y) * silu_f(ldf(z[k]))};
        stv<AT, 1>(a.out, t * inner + c, o1);
      }
      if (vec) {
#pragma unroll
        for (int i = 0; i < NS; i += 4)
          if (n0 + i < N) stv<float, 4>(st, (int64_t)c * N + n0 + i, &S[k][i]);
      } else {
#pragma unroll
        for (int i = 0; i < NS; ++i)
          if (n0 + i < N) st[(int64_t)c * N + n0 + i] = S[k][i];
      }
    }
  }
}

template <typename AT>
int selective_scan_t(const SelArgs<AT>& a, int S, bool one, cudaStream_t s) {
  const int N = a.n_state;
  const int vec = N % 4 == 0 && a.slot_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(a.state) | reinterpret_cast<uintptr_t>(a.A)) % 16 == 0;
#define SEL(LV, NV)                                                                                                                              \
  do {                                                                                                                                           \
    constexpr int CH = kSelThreads / LV, KB = 16 / NV;                                                                                            \
    if (one) B200_CUDA(launch(selective_step_kernel<AT, LV, NV, KB>, dim3(S, (a.inner + CH * KB - 1) / (CH * KB)), dim3(kSelThreads), (size_t)0, s, a, vec)); \
    else B200_CUDA(launch(selective_scan_kernel<AT, LV, NV>, dim3(S, (a.inner + CH - 1) / CH), dim3(kSelThreads), (size_t)0, s, a));              \
  } while (0)
  if (N <= 4) SEL(1, 4);
  else if (N <= 8) SEL(2, 4);
  else if (N <= 16) SEL(4, 4);
  else if (N <= 32) SEL(8, 4);
  else if (N <= 64) SEL(16, 4);
  else if (N <= 128) SEL(32, 4);
  else SEL(32, 8);
#undef SEL
  return B200_OK;
}

}  // namespace

int conv_inputs(bool f32, const void* fused, int64_t ld, const float* conv_a, int taps_a, float* tails_a, const float* conv_x, const float* bias_x,
                int taps_x, float* tails_x, int64_t slot_stride, const int32_t* positions, const int32_t* row_to_seq, const int32_t* seq_start,
                const int32_t* seq_slots, const int32_t* slots, float* qout, void* kc, void* vc, void* xc, int T, int heads, int kv_heads,
                int dim, int vdim, int inner, int block_size, bool one_row, cudaStream_t s, bool silu_x) {
  if (T == 0) return B200_OK;
  B200_REQUIRE(taps_a <= 1 || (conv_a && tails_a && seq_slots), B200_ERR_INVALID, "conv_inputs: the q/k/v convolution needs its weights and tails");
  B200_REQUIRE(inner == 0 || (taps_x >= 1 && conv_x && xc && (taps_x == 1 || (tails_x && seq_slots))), B200_ERR_INVALID,
               "conv_inputs: the second convolution needs its weights, tails and output");
  B200_REQUIRE(positions && seq_start && (heads == 0 || (slots && qout && kc && vc)), B200_ERR_INVALID, "conv_inputs: null argument");
  if (f32) {
    ConvArgs<float> a = {(const float*)fused, ld, conv_a, conv_x, bias_x, tails_a, tails_x, taps_a, taps_x, slot_stride, positions, row_to_seq, seq_start,
                         seq_slots, slots, qout, (float*)kc, (float*)vc, (float*)xc, T, heads, kv_heads, dim, vdim, inner, block_size,
                         one_row ? 1 : 0, 1, 0, silu_x ? 1 : 0};
    return conv_inputs_t<float>(a, s);
  }
  ConvArgs<__nv_bfloat16> a = {(const __nv_bfloat16*)fused, ld, conv_a, conv_x, bias_x, tails_a, tails_x, taps_a, taps_x, slot_stride, positions, row_to_seq,
                               seq_start, seq_slots, slots, qout, (__nv_bfloat16*)kc, (__nv_bfloat16*)vc, (__nv_bfloat16*)xc, T, heads, kv_heads, dim,
                               vdim, inner, block_size, one_row ? 1 : 0, 1, 0, silu_x ? 1 : 0};
  return conv_inputs_t<__nv_bfloat16>(a, s);
}

// rows of W_x's product: dt | B | C, dt and the total padded to multiples of 8 so that both matrix products can be addressed by TMA
int selective_dt_pad(int rank) { return (rank + 7) / 8 * 8; }
int selective_rows(int rank, int state) { return (selective_dt_pad(rank) + 2 * state + 7) / 8 * 8; }

int selective_scan(bool f32, const void* xc, const void* bc, int64_t ldbc, int b_off, const float* dt_pre, const float* dt_bias, const float* A,
                   const float* D, const void* z, int64_t ldz, const int32_t* positions, const int32_t* seq_start, const int32_t* seq_slots,
                   float* state, int64_t slot_stride, void* out, int S, int inner, int n_state, bool one_row, cudaStream_t s) {
  if (S == 0) return B200_OK;
  B200_REQUIRE(inner > 0 && n_state > 0 && n_state <= 256, B200_ERR_UNSUPPORTED, "selective_scan: %d channels, %d states (at most 256)", inner, n_state);
  if (f32) {
    SelArgs<float> a = {(const float*)xc, (const float*)bc, (const float*)z, ldbc, ldz, slot_stride, b_off, dt_pre, dt_bias, A, D, positions, seq_start,
                        seq_slots, state, (float*)out, inner, n_state};
    return selective_scan_t<float>(a, S, one_row, s);
  }
  SelArgs<__nv_bfloat16> a = {(const __nv_bfloat16*)xc, (const __nv_bfloat16*)bc, (const __nv_bfloat16*)z, ldbc, ldz, slot_stride, b_off, dt_pre, dt_bias, A,
                              D, positions, seq_start, seq_slots, state, (__nv_bfloat16*)out, inner, n_state};
  return selective_scan_t<__nv_bfloat16>(a, S, one_row, s);
}

}  // namespace b200
