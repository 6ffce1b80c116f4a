// Retention (B200_MIXER_RETENTION): linear attention with one fixed decay per head.  The fused projection of a token is
// q | k | v | gate (heads*dim, heads*dim, heads*vdim, heads*vdim); per head and sequence the state is S [vdim][dim], fp32, in the
// sequence's state slot:
//   q, k turned by the position's angles on their leading rot_dims dimensions, k times dim^-1/2
//   S = decay S + v k^T;   o = S q;   out = o / rms(o) * silu(gate)
//
//  * retention_step: one CTA per (sequence, head) does all of it, for portions of a few rows (decode) and for shapes the chunk form
//    does not take.  A warp owns value columns, a lane the key channels lane, lane + 32, ...; rows come eight at a time through
//    shared memory.  The state is read ahead of the dependency wait (no launch of the same step before this one writes it), so
//    that its way from HBM hides behind the projection.
//  * retention_chunk: long portions, chunks of 64 rows in parallel on the tensor cores, three launches:
//      1. U_c = sum_i decay^(n-1-i) v_i k_i^T of every chunk and head;
//      2. per sequence and head, elementwise: the state ahead of every chunk, S <- decay^n S + U_c, and the final state;
//      3. o_i = decay^(i+1) S_c q_i + sum_{j<=i} decay^(i-j) (q_i . k_j) v_j, unit RMS, gate.
//    Products are bf16 mma with fp32 accumulators over SPLIT operands: an fp32 value goes in as hi + lo bf16 (about 16 bits of
//    mantissa), so rotated q and k, scores, decays and the state keep close to their fp32 values; v is exact in bf16.
//    Chunk items: sequence s of the step owns the items start_s / 64 + s, ..., a numbering that needs no prefix sum (ceil(n / 64)
//    items always fit ahead of the next sequence's first); unused items leave at once.
#include <algorithm>

#include "common.cuh"

namespace b200 {
namespace {

template <typename AT> __device__ __forceinline__ float ldx(const AT* p, int64_t i);
template <> __device__ __forceinline__ float ldx<float>(const float* p, int64_t i) { return p[i]; }
template <> __device__ __forceinline__ float ldx<__nv_bfloat16>(const __nv_bfloat16* p, int64_t i) { return __bfloat162float(p[i]); }
template <typename AT> __device__ __forceinline__ void stx(AT* p, int64_t i, float v);
template <> __device__ __forceinline__ void stx<float>(float* p, int64_t i, float v) { p[i] = v; }
template <> __device__ __forceinline__ void stx<__nv_bfloat16>(__nv_bfloat16* p, int64_t i, float v) { p[i] = __float2bfloat16_rn(v); }

struct RetRot {
  const float* table;   // [max_pos][2][half] or null
  int half, half_layout;
  int64_t max_pos;
};

__device__ __forceinline__ const float* rot_row(const RetRot& r, int pos) {
  const int64_t p = pos < 0 ? 0 : (pos >= r.max_pos ? r.max_pos - 1 : pos);
  return r.table ? r.table + p * 2 * r.half : nullptr;
}

constexpr int kRsRows = 8, kRsThreads = 256, kRsWarps = kRsThreads / 32;

// GRP groups of 4 value columns per warp are in registers at a time
template <typename AT, int DPL, int GRP>
__global__ void __launch_bounds__(kRsThreads)
retention_step_kernel(const AT* __restrict__ fused, int64_t ld, RetRot rot, const float* __restrict__ decay, const int32_t* __restrict__ positions,
                      const int32_t* __restrict__ seq_start, const int32_t* __restrict__ seq_slots, float* __restrict__ state, int64_t slot_stride,
                      AT* __restrict__ out, int heads, int dim, int vd, float eps, int max_rows) {
  extern __shared__ float sm[];
  float* sq = sm;                        // [rows][dim]
  float* sk = sq + kRsRows * dim;
  float* sv = sk + kRsRows * dim;        // [rows][vd]
  float* so = sv + kRsRows * vd;
  const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int start = seq_start[s], n_rows = seq_start[s + 1] - start;
  if (n_rows <= 0 || (max_rows > 0 && n_rows > max_rows)) {
    pdl_wait();
    return;
  }
  bool fresh = positions[start] == 0;
  float* st = state + (int64_t)seq_slots[s] * slot_stride + (int64_t)h * vd * dim;
  const float g = decay[h], kscale = 1.0f / sqrtf((float)dim);
  float S[GRP][4][DPL];
  auto load_state = [&](int jb) {
#pragma unroll
    for (int p = 0; p < GRP; ++p)
#pragma unroll
      for (int c = 0; c < 4; ++c)
#pragma unroll
        for (int i = 0; i < DPL; ++i) {
          const int j = jb + (p * kRsWarps + warp) * 4 + c, d = lane + 32 * i;
          S[p][c][i] = (!fresh && j < vd && d < dim) ? st[(int64_t)j * dim + d] : 0.f;
        }
  };
  load_state(0);
  bool loaded = true;
  pdl_wait();
  pdl_launch_dependents();
  const int hd = heads * dim, hv = heads * vd;
  for (int b0 = 0; b0 < n_rows; b0 += kRsRows) {
    const int nb = min(kRsRows, n_rows - b0);
    __syncthreads();   // the batch before has been consumed
    const int npair = dim - rot.half;   // per row: `half` turning pairs, then the rest one by one
    for (int e = tid; e < nb * npair; e += kRsThreads) {
      const int r = e / npair, i = e - r * npair;
      const int64_t t = start + b0 + r;
      const AT* q = fused + t * ld + (int64_t)h * dim;
      const AT* k = q + hd;
      if (i < rot.half) {
        const float* cs = rot_row(rot, positions[t]);
        const float c = cs[i], sn = cs[rot.half + i];
        const int i0 = rot.half_layout ? i : 2 * i, i1 = rot.half_layout ? i + rot.half : 2 * i + 1;
        const float qa = ldx<AT>(q, i0), qb = ldx<AT>(q, i1), ka = ldx<AT>(k, i0), kb = ldx<AT>(k, i1);
        sq[r * dim + i0] = fmaf(qa, c, -qb * sn);
        sq[r * dim + i1] = fmaf(qb, c, qa * sn);
        sk[r * dim + i0] = fmaf(ka, c, -kb * sn) * kscale;
        sk[r * dim + i1] = fmaf(kb, c, ka * sn) * kscale;
      } else {
        const int d = i + rot.half;
        sq[r * dim + d] = ldx<AT>(q, d);
        sk[r * dim + d] = ldx<AT>(k, d) * kscale;
      }
    }
    for (int e = tid; e < nb * vd; e += kRsThreads) {
      const int r = e / vd, j = e - r * vd;
      sv[e] = ldx<AT>(fused, (start + b0 + r) * ld + 2 * hd + (int64_t)h * vd + j);
    }
    __syncthreads();
    for (int jb = 0; jb < vd; jb += GRP * kRsWarps * 4) {
      if (!loaded) load_state(jb);
      loaded = false;
      for (int r = 0; r < nb; ++r) {
        float q[DPL], k[DPL];
#pragma unroll
        for (int i = 0; i < DPL; ++i) {
          const int d = lane + 32 * i;
          q[i] = d < dim ? sq[r * dim + d] : 0.f;
          k[i] = d < dim ? sk[r * dim + d] : 0.f;
        }
        float acc[GRP * 4];
#pragma unroll
        for (int p = 0; p < GRP; ++p)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const int j = jb + (p * kRsWarps + warp) * 4 + c;
            const float v = j < vd ? sv[r * vd + j] : 0.f;
            float a = 0.f;
#pragma unroll
            for (int i = 0; i < DPL; ++i) {
              S[p][c][i] = fmaf(g, S[p][c][i], k[i] * v);
              a = fmaf(S[p][c][i], q[i], a);
            }
            acc[p * 4 + c] = a;
          }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
          for (int x = 0; x < GRP * 4; ++x) acc[x] += __shfl_xor_sync(0xffffffffu, acc[x], o);
#pragma unroll
        for (int x = 0; x < GRP * 4; ++x) {
          const int j = jb + ((x / 4) * kRsWarps + warp) * 4 + x % 4;
          if (lane == x && j < vd) so[r * vd + j] = acc[x];
        }
      }
#pragma unroll
      for (int p = 0; p < GRP; ++p)
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < DPL; ++i) {
            const int j = jb + (p * kRsWarps + warp) * 4 + c, d = lane + 32 * i;
            if (j < vd && d < dim) st[(int64_t)j * dim + d] = S[p][c][i];
          }
    }
    fresh = false;
    __syncthreads();
    for (int r = warp; r < nb; r += kRsWarps) {
      float ss = 0.f;
      for (int j = lane; j < vd; j += 32) ss = fmaf(so[r * vd + j], so[r * vd + j], ss);
      ss = warp_sum(ss);
      const float inv = 1.0f / sqrtf(ss / (float)vd + eps);
      const int64_t t = start + b0 + r;
      for (int j = lane; j < vd; j += 32) {
        const float z = ldx<AT>(fused, t * ld + 2 * hd + hv + (int64_t)h * vd + j);
        stx<AT>(out, t * hv + (int64_t)h * vd + j, so[r * vd + j] * inv * (z / (1.0f + expf(-z))));
      }
    }
  }
}

// ---- chunk form ----------------------------------------------------------------------------------------------------------------
constexpr int kRc = 64, kRcThreads = 256, kRcWarps = 8;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// the pair (a, b) as two bf16 pairs hi + lo
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - bf16lo(hi), b - bf16hi(hi));
}

// decay^0 .. decay^64 by repeated squaring in fp64, rounded once
__device__ __forceinline__ void fill_powers(float* pw, float decay) {
  for (int n = threadIdx.x; n <= kRc; n += blockDim.x) {
    double r = 1.0, b = (double)decay;
    for (int e = n; e; e >>= 1, b *= b)
      if (e & 1) r *= b;
    pw[n] = (float)r;
  }
}

// item -> (sequence, first row, rows): false for items nobody owns.  Every warp finds it on its own.
__device__ __forceinline__ bool chunk_item(const int32_t* __restrict__ seq_start, int S, int item, int min_rows, int& row0, int& n) {
  int best = -1;
  for (int s = threadIdx.x & 31; s < S; s += 32)
    if (seq_start[s] / kRc + s <= item) best = s;   // the bases rise with s
  best = __reduce_max_sync(0xffffffffu, best);
  if (best < 0) return false;
  const int start = seq_start[best], rows = seq_start[best + 1] - start, c = item - (start / kRc + best);
  if (rows <= min_rows || c * kRc >= rows) return false;
  row0 = start + c * kRc;
  n = min(kRc, rows - c * kRc);
  return true;
}

// eight fp32 values as eight bf16 hi and eight bf16 lo
__device__ __forceinline__ void split8(const float (&v)[8], __nv_bfloat16* hi, __nv_bfloat16* lo) {
  uint32_t h[4], l[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) split2(v[2 * i], v[2 * i + 1], h[i], l[i]);
  *reinterpret_cast<uint4*>(hi) = make_uint4(h[0], h[1], h[2], h[3]);
  *reinterpret_cast<uint4*>(lo) = make_uint4(l[0], l[1], l[2], l[3]);
}
__device__ __forceinline__ void unpack8(const uint4& u, float (&v)[8]) {
  v[0] = bf16lo(u.x), v[1] = bf16hi(u.x), v[2] = bf16lo(u.y), v[3] = bf16hi(u.y);
  v[4] = bf16lo(u.z), v[5] = bf16hi(u.z), v[6] = bf16lo(u.w), v[7] = bf16hi(u.w);
}
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
}

// rows row0 .. row0 + n - 1 of q or k (col: first column of the head) turned, times mul (and falling: times pw[n - 1 - row]) -> hi and lo
// tiles [64][dim + 8].  rot.half a multiple of 8: eight neighbouring entries and their partners at a time; else two.
__device__ __forceinline__ void stage_rotated(const __nv_bfloat16* __restrict__ fused, int64_t ld, int64_t col, const RetRot& rot,
                                              const int32_t* __restrict__ positions, int row0, int n, int dim, float mul, const float* pw, bool falling,
                                              __nv_bfloat16* hi, __nv_bfloat16* lo) {
  const int ks = dim + 8;
  if (rot.half % 8 == 0) {
    const int hp = rot.half / 8, per = hp + (dim - 2 * rot.half) / 8;
#pragma unroll 2
    for (int e = threadIdx.x; e < kRc * per; e += (int)blockDim.x) {
      const int r = e / per, p = e - r * per;
      const bool live = r < n;
      const __nv_bfloat16* src = fused + (int64_t)(row0 + (live ? r : 0)) * ld + col;
      const float m = live ? mul * (falling ? pw[n - 1 - r] : 1.0f) : 0.f;
      if (p < hp) {
        const int i = 8 * p;
        const float* cs = rot_row(rot, positions[row0 + (live ? r : 0)]);
        const uint4 ua = *reinterpret_cast<const uint4*>(src + i), ub = *reinterpret_cast<const uint4*>(src + i + rot.half);
        float c[8], sn[8], a[8], b[8], x[8], y[8];
        load8(cs + i, c);
        load8(cs + rot.half + i, sn);
        unpack8(ua, a);
        unpack8(ub, b);
#pragma unroll
        for (int v = 0; v < 8; ++v) {
          x[v] = fmaf(a[v], c[v], -b[v] * sn[v]) * m;
          y[v] = fmaf(b[v], c[v], a[v] * sn[v]) * m;
        }
        split8(x, hi + r * ks + i, lo + r * ks + i);
        split8(y, hi + r * ks + i + rot.half, lo + r * ks + i + rot.half);
      } else {
        const int i = 2 * rot.half + 8 * (p - hp);
        float a[8];
        unpack8(*reinterpret_cast<const uint4*>(src + i), a);
#pragma unroll
        for (int v = 0; v < 8; ++v) a[v] *= m;
        split8(a, hi + r * ks + i, lo + r * ks + i);
      }
    }
    return;
  }
  const int hp = rot.half / 2, per = hp + (dim - 2 * rot.half) / 2;
  for (int e = threadIdx.x; e < kRc * per; e += (int)blockDim.x) {
    const int r = e / per, p = e - r * per;
    const bool live = r < n;
    const __nv_bfloat16* src = fused + (int64_t)(row0 + (live ? r : 0)) * ld + col;
    const float m = live ? mul * (falling ? pw[n - 1 - r] : 1.0f) : 0.f;
    uint32_t h2, l2;
    if (p < hp) {
      const int i = 2 * p;
      const float* cs = rot_row(rot, positions[row0 + (live ? r : 0)]);
      const float2 c = *reinterpret_cast<const float2*>(cs + i), sn = *reinterpret_cast<const float2*>(cs + rot.half + i);
      const uint32_t ua = *reinterpret_cast<const uint32_t*>(src + i), ub = *reinterpret_cast<const uint32_t*>(src + i + rot.half);
      const float a0 = bf16lo(ua), a1 = bf16hi(ua), b0 = bf16lo(ub), b1 = bf16hi(ub);
      split2(fmaf(a0, c.x, -b0 * sn.x) * m, fmaf(a1, c.y, -b1 * sn.y) * m, h2, l2);
      *reinterpret_cast<uint32_t*>(hi + r * ks + i) = h2;
      *reinterpret_cast<uint32_t*>(lo + r * ks + i) = l2;
      split2(fmaf(b0, c.x, a0 * sn.x) * m, fmaf(b1, c.y, a1 * sn.y) * m, h2, l2);
      *reinterpret_cast<uint32_t*>(hi + r * ks + i + rot.half) = h2;
      *reinterpret_cast<uint32_t*>(lo + r * ks + i + rot.half) = l2;
    } else {
      const int i = 2 * rot.half + 2 * (p - hp);
      const uint32_t ua = *reinterpret_cast<const uint32_t*>(src + i);
      split2(bf16lo(ua) * m, bf16hi(ua) * m, h2, l2);
      *reinterpret_cast<uint32_t*>(hi + r * ks + i) = h2;
      *reinterpret_cast<uint32_t*>(lo + r * ks + i) = l2;
    }
  }
}

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst)), "l"(src));
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// value rows [64][vd + 8], zero past n (asynchronously: cp_async_wait_all before the barrier that opens the tile)
__device__ __forceinline__ void stage_values(const __nv_bfloat16* __restrict__ fused, int64_t ld, int64_t col, int row0, int n, int vd, __nv_bfloat16* vs) {
  const int per = vd / 8;
  for (int e = threadIdx.x; e < kRc * per; e += (int)blockDim.x) {
    const int r = e / per, p = e - r * per;
    __nv_bfloat16* dst = vs + r * (vd + 8) + 8 * p;
    if (r < n) cp_async16(dst, fused + (int64_t)(row0 + r) * ld + col + 8 * p);
    else *reinterpret_cast<uint4*>(dst) = make_uint4(0u, 0u, 0u, 0u);
  }
}

// 1. U[j][d] = sum_i v_i[j] decay^(n-1-i) k_i[d]
__global__ void __launch_bounds__(kRcThreads)
retention_chunk_state_kernel(const __nv_bfloat16* __restrict__ fused, int64_t ld, RetRot rot, const float* __restrict__ decay,
                             const int32_t* __restrict__ positions, const int32_t* __restrict__ seq_start, int n_seqs, int min_rows,
                             float* __restrict__ ws, int heads, int dim, int vd) {
  extern __shared__ __align__(16) unsigned char smraw[];
  __shared__ float pw[kRc + 1];
  pdl_wait();
  pdl_launch_dependents();
  const int item = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int row0, n;
  if (!chunk_item(seq_start, n_seqs, item, min_rows, row0, n)) return;
  const int ks = dim + 8, vs = vd + 8;
  __nv_bfloat16* Kh = reinterpret_cast<__nv_bfloat16*>(smraw);   // [64][ks]
  __nv_bfloat16* Kl = Kh + kRc * ks;
  __nv_bfloat16* Vs = Kl + kRc * ks;                             // [64][vs]
  fill_powers(pw, decay[h]);
  __syncthreads();
  stage_values(fused, ld, (int64_t)2 * heads * dim + (int64_t)h * vd, row0, n, vd, Vs);
  stage_rotated(fused, ld, (int64_t)(heads + h) * dim, rot, positions, row0, n, dim, 1.0f / sqrtf((float)dim), pw, true, Kh, Kl);
  cp_async_wait_all();
  __syncthreads();
  float* U = ws + ((int64_t)item * heads + h) * vd * dim;
  // a warp takes a strip of 16 value columns x 64 key channels
  const int nd = (dim + 63) / 64, strips = (vd / 16) * nd;
  for (int x = warp; x < strips; x += kRcWarps) {
    const int m0 = (x / nd) * 16, d0 = (x % nd) * 64, pairs = min(4, (dim - d0) / 16);
    float c[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) c[i][j] = 0.f;
#pragma unroll
    for (int k0 = 0; k0 < kRc; k0 += 16) {
      uint32_t a[4];
      ldsm_x4_t(a, Vs + (k0 + (lane >> 4) * 8 + (lane & 7)) * vs + m0 + ((lane >> 3) & 1) * 8);
      const int off = (k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * ks + d0 + (lane >> 4) * 8;
#pragma unroll
      for (int p = 0; p < 4; ++p)
        if (p < pairs) {
          uint32_t b[4];
          ldsm_x4_t(b, Kh + off + p * 16);
          mma_bf16(c[2 * p], a, b[0], b[1]);
          mma_bf16(c[2 * p + 1], a, b[2], b[3]);
          ldsm_x4_t(b, Kl + off + p * 16);
          mma_bf16(c[2 * p], a, b[0], b[1]);
          mma_bf16(c[2 * p + 1], a, b[2], b[3]);
        }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i < 2 * pairs) {
        const int j = m0 + (lane >> 2), d = d0 + i * 8 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(U + (int64_t)j * dim + d) = make_float2(c[i][0], c[i][1]);
        *reinterpret_cast<float2*>(U + (int64_t)(j + 8) * dim + d) = make_float2(c[i][2], c[i][3]);
      }
  }
}

// 2. elementwise over the state: U_c becomes, in place, the state ahead of chunk c as bf16 (blocks of 8 hi, then their 8 lo); the last
// state goes into the slot.  Two neighbouring threads share a block: both have read it before either writes.
__global__ void __launch_bounds__(128)
retention_chunk_scan_kernel(const float* __restrict__ decay, const int32_t* __restrict__ positions, const int32_t* __restrict__ seq_start,
                            const int32_t* __restrict__ seq_slots, int min_rows, float* __restrict__ ws, float* __restrict__ state, int64_t slot_stride,
                            int heads, int elems) {
  pdl_wait();
  pdl_launch_dependents();
  const int s = blockIdx.x, h = blockIdx.y, e = (blockIdx.z * 128 + threadIdx.x) * 4;
  const int start = seq_start[s], rows = seq_start[s + 1] - start;
  if (rows <= min_rows || e >= elems) return;
  float* st = state + (int64_t)seq_slots[s] * slot_stride + (int64_t)h * elems + e;
  float4 S = positions[start] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st);
  const int chunks = (rows + kRc - 1) / kRc;
  float* U = ws + ((int64_t)(start / kRc + s) * heads + h) * elems + e;
  const int64_t stride = (int64_t)heads * elems;
  double full = (double)decay[h];
#pragma unroll
  for (int i = 0; i < 6; ++i) full *= full;   // decay^64
  const float gf = (float)full;
  constexpr int kAhead = 8;   // chunk loads in flight
  for (int c0 = 0; c0 < chunks; c0 += kAhead) {
    float4 u[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
      if (c0 + i < chunks) u[i] = *reinterpret_cast<const float4*>(U + (c0 + i) * stride);
    __syncwarp();   // the blocks are shared with a neighbouring thread (whole warps are in range: elems is a multiple of 256)
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      const int c = c0 + i;
      if (c >= chunks) break;
      float g = gf;
      const int n = rows - c * kRc;
      if (n < kRc) {
        double r = 1.0, b = (double)decay[h];
        for (int x = n; x; x >>= 1, b *= b)
          if (x & 1) r *= b;
        g = (float)r;
      }
      uint32_t h0, l0, h1, l1;
      split2(S.x, S.y, h0, l0);
      split2(S.z, S.w, h1, l1);
      // U points at element e: back to the block of 8, then this thread's half of its hi and of its lo
      __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(U - (e & 4) + c * stride) + (e & 4);
      *reinterpret_cast<uint2*>(dst) = make_uint2(h0, h1);
      *reinterpret_cast<uint2*>(dst + 8) = make_uint2(l0, l1);
      S = make_float4(fmaf(g, S.x, u[i].x), fmaf(g, S.y, u[i].y), fmaf(g, S.z, u[i].z), fmaf(g, S.w, u[i].w));
    }
  }
  *reinterpret_cast<float4*>(st) = S;
}

// 3. outputs of a chunk.  Warp w: rows 16 (w & 3) ..; quarter w >> 2 takes 16 of the 64 keys (scores) and every fourth group of 16 value
// columns (outputs).
constexpr int kRoThreads = 512;
__global__ void __launch_bounds__(kRoThreads)
retention_chunk_out_kernel(const __nv_bfloat16* __restrict__ fused, int64_t ld, RetRot rot, const float* __restrict__ decay,
                           const int32_t* __restrict__ positions, const int32_t* __restrict__ seq_start, int n_seqs, int min_rows,
                           const float* __restrict__ ws, __nv_bfloat16* __restrict__ out, int heads, int dim, int vd, float eps) {
  extern __shared__ __align__(16) unsigned char smraw[];
  __shared__ float pw[kRc + 1];
  __shared__ float ssq[4][kRc];
  pdl_wait();
  pdl_launch_dependents();
  const int item = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int row0, n;
  if (!chunk_item(seq_start, n_seqs, item, min_rows, row0, n)) return;
  const int ks = dim + 8, vs = vd + 8, ps = kRc + 8;
  __nv_bfloat16* Qh = reinterpret_cast<__nv_bfloat16*>(smraw);   // [64][ks]
  __nv_bfloat16* Ql = Qh + kRc * ks;
  __nv_bfloat16* Kh = Ql + kRc * ks;
  __nv_bfloat16* Kl = Kh + kRc * ks;
  __nv_bfloat16* Vs = Kl + kRc * ks;                             // [64][vs]
  __nv_bfloat16* Sh = Vs + kRc * vs;                             // [vd][ks]
  __nv_bfloat16* Sl = Sh + vd * ks;
  __nv_bfloat16* Ph = Sl + vd * ks;                              // [64][ps]
  __nv_bfloat16* Pl = Ph + kRc * ps;
  const __nv_bfloat16* U = reinterpret_cast<const __nv_bfloat16*>(ws + ((int64_t)item * heads + h) * vd * dim);
  const int per_s = dim / 8;
  for (int e = threadIdx.x; e < vd * per_s; e += kRoThreads) {
    const int j = e / per_s, d = (e - j * per_s) * 8;
    cp_async16(Sh + j * ks + d, U + (int64_t)e * 16);
    cp_async16(Sl + j * ks + d, U + (int64_t)e * 16 + 8);
  }
  stage_values(fused, ld, (int64_t)2 * heads * dim + (int64_t)h * vd, row0, n, vd, Vs);
  stage_rotated(fused, ld, (int64_t)h * dim, rot, positions, row0, n, dim, 1.0f, pw, false, Qh, Ql);
  stage_rotated(fused, ld, (int64_t)(heads + h) * dim, rot, positions, row0, n, dim, 1.0f / sqrtf((float)dim), pw, false, Kh, Kl);
  fill_powers(pw, decay[h]);
  __syncthreads();
  const int r0 = (warp & 3) * 16, quarter = warp >> 2;
  const int rl = r0 + (lane >> 2);   // this lane's rows: rl and rl + 8
  const int qoff = (r0 + (lane & 15)) * ks + (lane >> 4) * 8;
  const int boff = (lane & 7) + (lane >> 4) * 8, bcol = ((lane >> 3) & 1) * 8;   // two 8-row groups of a B operand stored [n][k]
  {
    // scores of 16 rows against keys 16 quarter .. + 15; the three split products have accumulators of their own
    float c[3][2][4];
#pragma unroll
    for (int x = 0; x < 3; ++x)
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) c[x][i][j] = 0.f;
    const int key0 = quarter * 16;
    if (key0 <= r0) {
#pragma unroll 2
      for (int k0 = 0; k0 < dim; k0 += 16) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        ldsm_x4(ah, Qh + qoff + k0);
        ldsm_x4(bh, Kh + (key0 + boff) * ks + k0 + bcol);
        ldsm_x4(al, Ql + qoff + k0);
        ldsm_x4(bl, Kl + (key0 + boff) * ks + k0 + bcol);
        mma_bf16(c[0][0], ah, bh[0], bh[1]);
        mma_bf16(c[0][1], ah, bh[2], bh[3]);
        mma_bf16(c[1][0], al, bh[0], bh[1]);
        mma_bf16(c[1][1], al, bh[2], bh[3]);
        mma_bf16(c[2][0], ah, bl[0], bl[1]);
        mma_bf16(c[2][1], ah, bl[2], bl[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int key = key0 + i * 8 + (lane & 3) * 2;
#pragma unroll
      for (int hr = 0; hr < 2; ++hr) {
        const int r = rl + hr * 8;
        const float s0 = c[0][i][2 * hr] + (c[1][i][2 * hr] + c[2][i][2 * hr]);
        const float s1 = c[0][i][2 * hr + 1] + (c[1][i][2 * hr + 1] + c[2][i][2 * hr + 1]);
        uint32_t h2, l2;
        split2(key <= r ? s0 * pw[r - key] : 0.f, key + 1 <= r ? s1 * pw[r - key - 1] : 0.f, h2, l2);
        *reinterpret_cast<uint32_t*>(Ph + r * ps + key) = h2;
        *reinterpret_cast<uint32_t*>(Pl + r * ps + key) = l2;
      }
    }
  }
  cp_async_wait_all();
  __syncthreads();   // every quarter's scores, the values and the state are in place
  // up to two groups of 16 value columns: the state's part first
  float o[2][2][4];
#pragma unroll
  for (int u = 0; u < 2; ++u)
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) o[u][i][j] = 0.f;
  const int n_units = vd / 16;
#pragma unroll 2
  for (int k0 = 0; k0 < dim; k0 += 16) {
    uint32_t ah[4], al[4];
    ldsm_x4(ah, Qh + qoff + k0);
    ldsm_x4(al, Ql + qoff + k0);
#pragma unroll
    for (int u = 0; u < 2; ++u)
      if (quarter + 4 * u < n_units) {
        uint32_t bh[4], bl[4];
        const int jr = (quarter + 4 * u) * 16 + boff;
        ldsm_x4(bh, Sh + jr * ks + k0 + bcol);
        ldsm_x4(bl, Sl + jr * ks + k0 + bcol);
        mma_bf16(o[u][0], al, bh[0], bh[1]);
        mma_bf16(o[u][1], al, bh[2], bh[3]);
        mma_bf16(o[u][0], ah, bl[0], bl[1]);
        mma_bf16(o[u][1], ah, bl[2], bl[3]);
        mma_bf16(o[u][0], ah, bh[0], bh[1]);
        mma_bf16(o[u][1], ah, bh[2], bh[3]);
      }
  }
  {
    const float d0 = pw[rl + 1], d1 = pw[rl + 9];
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int i = 0; i < 2; ++i) o[u][i][0] *= d0, o[u][i][1] *= d0, o[u][i][2] *= d1, o[u][i][3] *= d1;
  }
  for (int k0 = 0; k0 <= r0; k0 += 16) {   // keys past the warp's rows carry zero weight
    uint32_t ah[4], al[4];
    ldsm_x4(ah, Ph + (r0 + (lane & 15)) * ps + k0 + (lane >> 4) * 8);
    ldsm_x4(al, Pl + (r0 + (lane & 15)) * ps + k0 + (lane >> 4) * 8);
#pragma unroll
    for (int u = 0; u < 2; ++u)
      if (quarter + 4 * u < n_units) {
        uint32_t b[4];
        ldsm_x4_t(b, Vs + (k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * vs + (quarter + 4 * u) * 16 + (lane >> 4) * 8);
        mma_bf16(o[u][0], al, b[0], b[1]);
        mma_bf16(o[u][1], al, b[2], b[3]);
        mma_bf16(o[u][0], ah, b[0], b[1]);
        mma_bf16(o[u][1], ah, b[2], b[3]);
      }
  }
  float s0 = 0.f, s1 = 0.f;
#pragma unroll
  for (int u = 0; u < 2; ++u)
#pragma unroll
    for (int i = 0; i < 2; ++i) {   // a group that is not there holds zeros
      s0 = fmaf(o[u][i][0], o[u][i][0], fmaf(o[u][i][1], o[u][i][1], s0));
      s1 = fmaf(o[u][i][2], o[u][i][2], fmaf(o[u][i][3], o[u][i][3], s1));
    }
#pragma unroll
  for (int x = 1; x < 4; x <<= 1) {
    s0 += __shfl_xor_sync(0xffffffffu, s0, x);
    s1 += __shfl_xor_sync(0xffffffffu, s1, x);
  }
  if ((lane & 3) == 0) {
    ssq[quarter][rl] = s0;
    ssq[quarter][rl + 8] = s1;
  }
  __syncthreads();
  const int64_t hv = (int64_t)heads * vd;
#pragma unroll
  for (int hr = 0; hr < 2; ++hr) {
    const int r = rl + hr * 8;
    if (r >= n) continue;
    const float inv = 1.0f / sqrtf(((ssq[0][r] + ssq[1][r]) + (ssq[2][r] + ssq[3][r])) / (float)vd + eps);
    const __nv_bfloat16* gate = fused + (int64_t)(row0 + r) * ld + (int64_t)2 * heads * dim + hv + (int64_t)h * vd;
    __nv_bfloat16* dst = out + (int64_t)(row0 + r) * hv + (int64_t)h * vd;
#pragma unroll
    for (int u = 0; u < 2; ++u)
      if (quarter + 4 * u < n_units) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int j = (quarter + 4 * u) * 16 + i * 8 + (lane & 3) * 2;
          const uint32_t z2 = *reinterpret_cast<const uint32_t*>(gate + j);
          const float za = bf16lo(z2), zb = bf16hi(z2);
          *reinterpret_cast<uint32_t*>(dst + j) =
              pack_bf16(o[u][i][2 * hr] * inv * (za / (1.0f + expf(-za))), o[u][i][2 * hr + 1] * inv * (zb / (1.0f + expf(-zb))));
        }
      }
  }
}

size_t rc_state_smem(int dim, int vd) { return (size_t)kRc * (2 * (dim + 8) + vd + 8) * 2; }
size_t rc_out_smem(int dim, int vd) { return (size_t)kRc * (4 * (dim + 8) + vd + 8) * 2 + (size_t)2 * vd * (dim + 8) * 2 + (size_t)2 * kRc * (kRc + 8) * 2; }

template <typename AT>
int retention_step_t(const void* fused, int64_t ld, const RetRot& rot, const float* decay, const int32_t* positions, const int32_t* seq_start,
                     const int32_t* seq_slots, float* state, int64_t slot_stride, void* out, int S, int heads, int dim, int vd, float eps, int max_rows,
                     cudaStream_t s) {
  const size_t smem = (size_t)kRsRows * 2 * (dim + vd) * 4;
  B200_REQUIRE(smem <= 200 * 1024, B200_ERR_UNSUPPORTED, "retention: heads of %d x %d do not fit shared memory", dim, vd);
  const int dpl = (dim + 31) / 32;
#define RS(D, G)                                                                                                                          \
  do {                                                                                                                                    \
    static bool done[64] = {};                                                                                                            \
    if (smem > 48 * 1024) B200_CUDA(ensure_dynamic_smem(retention_step_kernel<AT, D, G>, 200 * 1024, done));                              \
    B200_CUDA(launch(retention_step_kernel<AT, D, G>, dim3(S, heads), dim3(kRsThreads), smem, s, (const AT*)fused, ld, rot, decay, positions, \
                     seq_start, seq_slots, state, slot_stride, (AT*)out, heads, dim, vd, eps, max_rows));                                 \
  } while (0)
#define RSG(D)            \
  do {                    \
    if (vd <= 32) RS(D, 1); \
    else if (vd <= 64) RS(D, 2); \
    else RS(D, (D <= 4 ? 4 : 2)); \
  } while (0)
  if (dpl <= 1) RSG(1);
  else if (dpl <= 2) RSG(2);
  else if (dpl <= 4) RSG(4);
  else RSG(8);
#undef RSG
#undef RS
  return B200_OK;
}

}  // namespace

int retention_step(bool f32, const void* fused, int64_t ld, const float* rot, int rot_dims, bool half_layout, int64_t max_pos,
                   const float* decay, const int32_t* positions, const int32_t* seq_start, const int32_t* seq_slots, float* state,
                   int64_t slot_stride, void* out, int S, int heads, int dim, int vdim, float eps, int max_rows, cudaStream_t s) {
  if (S == 0) return B200_OK;
  B200_REQUIRE(heads > 0 && dim > 0 && dim <= 256 && vdim > 0, B200_ERR_UNSUPPORTED, "retention: key size %d outside (0, 256]", dim);
  B200_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim, B200_ERR_INVALID, "retention: %d rotated dimensions in heads of %d", rot_dims, dim);
  const RetRot rr = {rot, rot ? rot_dims / 2 : 0, half_layout ? 1 : 0, max_pos};
  return f32 ? retention_step_t<float>(fused, ld, rr, decay, positions, seq_start, seq_slots, state, slot_stride, out, S, heads, dim, vdim, eps, max_rows, s)
             : retention_step_t<__nv_bfloat16>(fused, ld, rr, decay, positions, seq_start, seq_slots, state, slot_stride, out, S, heads, dim, vdim, eps,
                                               max_rows, s);
}

bool retention_chunk_supported(int dim, int vdim) {
  return dim > 0 && vdim > 0 && dim % 16 == 0 && vdim % 16 == 0 && dim <= 256 && vdim <= 128 && rc_out_smem(dim, vdim) <= 200 * 1024;
}

int64_t retention_chunk_workspace_bytes(int T, int S, int heads, int dim, int vdim) { return (int64_t)(T / kRc + S + 1) * heads * dim * vdim * 4; }

int retention_chunk(const void* fused, int64_t ld, const float* rot, int rot_dims, bool half_layout, int64_t max_pos, const float* decay,
                    const int32_t* positions, const int32_t* seq_start, const int32_t* seq_slots, float* state, int64_t slot_stride, void* out,
                    int T, int S, int heads, int dim, int vdim, float eps, int min_rows, void* ws, cudaStream_t s) {
  if (T == 0 || S == 0) return B200_OK;
  B200_REQUIRE(retention_chunk_supported(dim, vdim), B200_ERR_UNSUPPORTED, "retention_chunk: heads of %d x %d", dim, vdim);
  B200_REQUIRE(!rot || (half_layout && rot_dims % 4 == 0 && rot_dims <= dim), B200_ERR_UNSUPPORTED, "retention_chunk: %d rotated dimensions", rot_dims);
  B200_REQUIRE(ws && ld % 8 == 0 && reinterpret_cast<uintptr_t>(fused) % 16 == 0 && (!rot || reinterpret_cast<uintptr_t>(rot) % 16 == 0) && reinterpret_cast<uintptr_t>(state) % 16 == 0 && slot_stride % 4 == 0,
               B200_ERR_INVALID, "retention_chunk: misaligned operands or no workspace");
  const RetRot rr = {rot, rot ? rot_dims / 2 : 0, 1, max_pos};
  const __nv_bfloat16* f = (const __nv_bfloat16*)fused;
  const int items = T / kRc + S;
  const size_t sm1 = rc_state_smem(dim, vdim), sm3 = rc_out_smem(dim, vdim);
  static bool d1[64] = {}, d3[64] = {};
  if (sm1 > 48 * 1024) B200_CUDA(ensure_dynamic_smem(retention_chunk_state_kernel, 200 * 1024, d1));
  if (sm3 > 48 * 1024) B200_CUDA(ensure_dynamic_smem(retention_chunk_out_kernel, 200 * 1024, d3));
  B200_CUDA(launch(retention_chunk_state_kernel, dim3(items, heads), dim3(kRcThreads), sm1, s, f, ld, rr, decay, positions, seq_start, S, min_rows,
                   (float*)ws, heads, dim, vdim));
  const int elems = dim * vdim;
  B200_CUDA(launch(retention_chunk_scan_kernel, dim3(S, heads, (elems / 4 + 127) / 128), dim3(128), (size_t)0, s, decay, positions, seq_start, seq_slots,
                   min_rows, (float*)ws, state, slot_stride, heads, elems));
  B200_CUDA(launch(retention_chunk_out_kernel, dim3(items, heads), dim3(kRoThreads), sm3, s, f, ld, rr, decay, positions, seq_start, S, min_rows,
                   (const float*)ws, (__nv_bfloat16*)out, heads, dim, vdim, eps));
  return B200_OK;
}

}  // namespace b200
