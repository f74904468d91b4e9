// Gated linear attention.  Per head, with one decay a token and key channel:
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T;   o_t = S_t^T q_t;   a = sigmoid(W u + bias)^(1 / tau)
// Here are the kernels for many tokens of a sequence, chunk by chunk, and for a decode step, which has one token of every
// sequence (state_scan.cu walks the same recurrence token by token: short portions, and sizes that these do not take).
//
//   gla_decode          a block per (sequence, head): the state's rows are asked for first, all of a warp's at once; then the
//                       decays, the update, the read-out, the head's root mean square, its weight and the silu gate, in one
//                       kernel between the two projections
//
// Many tokens.  A chunk is C tokens of one
// sequence's rows of the step, from the step's first row on.  With b_t = ln a_1 + .. + ln a_t inside a chunk that starts at S:
//   o_t = S^T (exp(b_t) q_t) + sum_(s <= t) A[t, s] v_s         A[t, s] = sum_d q_t[d] k_s[d] a_(s+1)[d] .. a_t[d]
//   S'  = diag(exp(b_C)) S + sum_s (exp(b_C - b_s) k_s) v_s^T
// No exponent is ever positive, so nothing overflows however strong the decays are.  All of it is float32.
//
//   gla_chunk_prepare   a block per (chunk, head), no chunk waits for another: the decays (a channel a thread), exp(b_t) q_t,
//                       exp(b_C - b_s) k_s, exp(b_C), A (a thread per s and run of channels carries k_s times the running
//                       product of decays over t) and v, all in float32, as one contiguous record of fixed layout
//   gla_chunk_scan      a block per (sequence, head, run of value columns) walks the sequence's records with its part of S in
//                       registers: a thread holds 8 channels x 2 value columns, both products run on pairs of channels
//                       (fma.rn.f32x2), the column sums over channels go through a reduce-scatter of four lanes and
//                       shared memory; records come by bulk copies (cp.async.bulk on mbarriers), several chunks ahead
//
// Record (floats), DP = the key size rounded up to 32, 64, 128 or 256, VP = the value size rounded up to VB, rows beyond a chunk's tokens and
// columns beyond the sizes zero (decays one):
//   [exp(b) q: C x DP][exp(b_C - b) k: C x DP][exp(b_C): DP][A transposed, (s, t): C x C][v: VP / VB runs of C x VB]
#include "common.cuh"

namespace {
constexpr int C = 16;
constexpr int PREP_THREADS = 128;
constexpr int STAGES = 3;

__device__ __forceinline__ size_t record_floats(int DP, int VP) { return (size_t)2 * C * DP + DP + C * C + (size_t)C * VP; }

__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

// `bytes` of a row to shared memory, 16 at a time where `vec` (rows and sizes of 16 bytes), else value by value
__device__ __forceinline__ void copy16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
// n rows of `count` values (stride `stride`) into rows of `row` values, the rows beyond n up to C zero
template <typename T> __device__ __forceinline__ void stage_tile(T* dst, int row, const T* src, size_t stride, int n, int count, bool vec) {
  if (vec) {
    constexpr int PER = 16 / (int)sizeof(T);
    const int pieces = count / PER;
    for (int i = threadIdx.x; i < C * pieces; i += PREP_THREADS) {
      const int t = i / pieces, c = (i - t * pieces) * PER;
      if (t < n) copy16(dst + t * row + c, src + t * stride + c);
      else *reinterpret_cast<uint4*>(dst + t * row + c) = make_uint4(0, 0, 0, 0);
    }
  } else {
    for (int i = threadIdx.x; i < C * count; i += PREP_THREADS) {
      const int t = i / count, c = i - t * count;
      dst[t * row + c] = t < n ? src[t * stride + c] : from_f32<T>(0.f);
    }
  }
}

// chunk_rows [chunks, 2]: first row and end of every chunk.  w [heads * dim, rank], bias float32 [heads * dim].
template <typename T, typename TW>
__global__ void __launch_bounds__(PREP_THREADS) gla_chunk_prepare_kernel(const T* proj, int stride, int u_col, int rank, const TW* w,
                                                                         const float* bias, float inv_tau, const int* chunk_rows,
                                                                         float* records, int heads, int dim, int vdim, int DP,
                                                                         int VP, int VB, float q_scale, int n_tokens, int vec_qk,
                                                                         int vec_v) {
  extern __shared__ __align__(16) float sm[];
  const int KS = DP + 4;                // padded rows of k: threads of a warp read different ones
  float* qs = sm;                       // [C][DP]
  float* as = qs + C * DP;              // [C][DP]
  float* ks = as + C * DP;              // [C][KS]
  float* us = ks + C * KS;              // [C][rank], rank rounded up to 4
  const int RP = (rank + 3) & ~3, VR = (vdim + 7) & ~7;
  // no early launch of the kernel that follows: the scan has about a block a multiprocessor, and started while these blocks
  // still fill most of them, its blocks would crowd on the few that are free
  T* rq = reinterpret_cast<T*>(us + C * RP);  // the projection's values: [C][DP] of q, of k, [C][VR] of v
  T* rk = rq + C * DP;
  T* rv = rk + C * DP;
  pdl_wait();
  const int chunk = blockIdx.x, head = blockIdx.y, tid = threadIdx.x;
  const int r0 = __ldcg(chunk_rows + 2 * chunk), n = min(__ldcg(chunk_rows + 2 * chunk + 1) - r0, C);
  if (!FMS_IN(r0, n_tokens) || !FMS_IN(r0 + n - 1, n_tokens)) return;  // the whole block alike
  float* rec = records + ((size_t)chunk * heads + head) * record_floats(DP, VP);
  const T* qp = proj + (size_t)r0 * stride + (size_t)head * dim;
  stage_tile(rq, DP, qp, stride, n, dim, vec_qk);
  stage_tile(rk, DP, qp + (size_t)heads * dim, stride, n, dim, vec_qk);
  stage_tile(rv, VR, proj + (size_t)r0 * stride + 2 * (size_t)heads * dim + (size_t)head * vdim, stride, n, vdim, vec_v);
  for (int i = tid; i < C * RP; i += PREP_THREADS) {
    const int t = i / RP, r = i - t * RP;
    us[i] = t < n && r < rank ? to_f32(proj[(size_t)(r0 + t) * stride + u_col + r]) : 0.f;
  }
  asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;\n" ::: "memory");
  __syncthreads();
  for (int d = tid; d < DP; d += PREP_THREADS) {
    float b[C];  // ln a_t, then its sums
#pragma unroll
    for (int t = 0; t < C; ++t) b[t] = 0.f;
    if (d < dim) {
      const TW* row = w + ((size_t)head * dim + d) * rank;
      for (int r = 0; r < RP; r += 4) {
        float wv[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) wv[k] = r + k < rank ? to_f32(row[r + k]) : 0.f;
#pragma unroll
        for (int t = 0; t < C; ++t) {
          const float4 u = *reinterpret_cast<const float4*>(us + t * RP + r);
          b[t] = fmaf(wv[0], u.x, fmaf(wv[1], u.y, fmaf(wv[2], u.z, fmaf(wv[3], u.w, b[t]))));
        }
      }
      const float bd = bias[(size_t)head * dim + d];
#pragma unroll
      for (int t = 0; t < C; ++t) b[t] = t < n ? -softplus_f(-(b[t] + bd)) * inv_tau : 0.f;
    }
    float sum = 0.f;
#pragma unroll
    for (int t = 0; t < C; ++t) {
      as[t * DP + d] = expf(b[t]);
      sum += b[t];
      b[t] = sum;
      const float q = d < dim ? to_f32(rq[t * DP + d]) * q_scale : 0.f;
      qs[t * DP + d] = q;
      rec[t * DP + d] = q * expf(sum);
    }
#pragma unroll
    for (int t = 0; t < C; ++t) {
      const float k = d < dim ? to_f32(rk[t * DP + d]) : 0.f;
      ks[t * KS + d] = k;
      rec[(C + t) * DP + d] = k * expf(sum - b[t]);
    }
    rec[2 * C * DP + d] = expf(sum);
  }
  {  // v: runs of VB columns, each C x VB
    float* dst = rec + 2 * C * DP + DP + C * C;
    const int per = VP / 4, vb_log = VB == 32 ? 5 : 4;
    for (int i = tid; i < C * per; i += PREP_THREADS) {
      const int t = i / per, v = (i - t * per) * 4;
      float x[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) x[k] = v + k < vdim ? to_f32(rv[t * VR + v + k]) : 0.f;
      *reinterpret_cast<float4*>(dst + ((size_t)(v >> vb_log) * C + t) * VB + (v & (VB - 1))) = make_float4(x[0], x[1], x[2], x[3]);
    }
  }
  __syncthreads();
  // A: thread (s, run of channels); k_s carries the product of the decays after s
  const int s = tid & (C - 1), run = tid / C;  // 8 runs
  float acc[C];
#pragma unroll
  for (int t = 0; t < C; ++t) acc[t] = 0.f;
  for (int d = 4 * run; d < DP; d += 32) {
    float4 k = *reinterpret_cast<const float4*>(ks + s * KS + d);
#pragma unroll
    for (int t = 0; t < C; ++t) {
      const float4 q = *reinterpret_cast<const float4*>(qs + t * DP + d);
      const float4 a = *reinterpret_cast<const float4*>(as + t * DP + d);
      if (t > s) k.x *= a.x, k.y *= a.y, k.z *= a.z, k.w *= a.w;
      if (t >= s) acc[t] = fmaf(q.x, k.x, fmaf(q.y, k.y, fmaf(q.z, k.z, fmaf(q.w, k.w, acc[t]))));
    }
  }
  __syncthreads();  // qs is free
  float* red = qs;  // [4 warps][C s][C t]
#pragma unroll
  for (int t = 0; t < C; ++t) {
    acc[t] += __shfl_xor_sync(0xffffffffu, acc[t], 16);
    if ((tid & 31) < 16) red[((tid >> 5) * C + s) * C + t] = acc[t];
  }
  __syncthreads();
  float* at = rec + 2 * C * DP + DP;
  for (int i = tid; i < C * C; i += PREP_THREADS) at[i] = (red[i] + red[C * C + i]) + (red[2 * C * C + i] + red[3 * C * C + i]);
}

// ---- the scan over chunks ------------------------------------------------------------------------------
typedef unsigned long long f32x2;  // two floats side by side in registers
__device__ __forceinline__ f32x2 pack2(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};\n" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;\n" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;\n" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;\n" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
struct Eight {
  f32x2 p[4];
};
__device__ __forceinline__ Eight load8(const float* x) {  // shared memory, 16-byte aligned
  Eight e;
  const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(x), b = *reinterpret_cast<const ulonglong2*>(x + 4);
  e.p[0] = a.x, e.p[1] = a.y, e.p[2] = b.x, e.p[3] = b.y;
  return e;
}

// Block: WD = DP / 32 warps along the channels x VB / 16 along the value columns.  A lane holds channels d0 .. d0 + 8 of
// columns v0, v0 + 1.  state [slots, heads, vdim, dim]; o [tokens, heads * vdim].
template <int DP, int VB>
__global__ void __launch_bounds__(DP / 32 * (VB / 16) * 32) gla_chunk_scan_kernel(const float* records, const int* chunk_rows, const int* first_chunk,
                                                             float* state, float* o, const int* slots, int heads, int dim, int vdim,
                                                             int VP, int write_state, int n_slots, int n_tokens,
                                                             int* error_flag) {
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(8) unsigned long long full[STAGES];
  pdl_launch_dependents();
  const int seq = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  constexpr int WD = DP / 32;
  const int wd = warp % WD, wv = warp / WD;
  const int dgl = lane >> 3, vgl = lane & 7, dg = wd * 4 + dgl;
  const int d0 = dg * 8, vl = wv * 16 + vgl * 2, v0 = blockIdx.z * VB + vl;
  constexpr int head_part = 2 * C * DP + DP + C * C, stage_floats = head_part + C * VB;
  float* red = sm + STAGES * stage_floats;  // [2][WD][C][VB]
  if (tid == 0) {
    for (int i = 0; i < STAGES; ++i) mbar_init(full + i, 1);
    mbar_fence_init();
  }
  pdl_wait();
  const int slot = __ldcg(slots + seq);
  if (!FMS_IN(slot, n_slots)) return;  // the whole block alike
  const int c_lo = __ldcg(first_chunk + seq), c_hi = __ldcg(first_chunk + seq + 1);
  const size_t rec_floats = record_floats(DP, VP);
  const int first_row = c_lo < c_hi ? __ldcg(chunk_rows + 2 * c_lo) : 0;  // a sequence's chunks follow one another
  const int end_row = c_lo < c_hi ? __ldcg(chunk_rows + 2 * c_hi - 1) : 0;
  auto issue = [&](int c) {  // one thread
    const int st = (c - c_lo) % STAGES;
    const float* rec = records + ((size_t)c * heads + head) * rec_floats;
    float* dst = sm + st * stage_floats;
    mbar_arrive_expect_tx(full + st, (uint32_t)(stage_floats * sizeof(float)));
    bulk_copy_g2s(dst, rec, (uint32_t)(head_part * sizeof(float)), full + st);
    bulk_copy_g2s(dst + head_part, rec + head_part + (size_t)blockIdx.z * C * VB, (uint32_t)(C * VB * sizeof(float)), full + st);
  };
  __syncthreads();
  if (tid == 0)
    for (int c = c_lo; c < min(c_hi, c_lo + STAGES); ++c) issue(c);
  f32x2 S[4][2];  // [pair of channels][column]
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const float* p = state + (((size_t)slot * heads + head) * vdim + min(v0 + i, vdim - 1)) * dim;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = d0 + 2 * j;
      const bool in = v0 + i < vdim;
      S[j][i] = pack2(in && d < dim ? p[d] : 0.f, in && d + 1 < dim ? p[d + 1] : 0.f);
    }
  }
  bool dead = false;  // a copy did not come in time: the block goes on with what lies there, and says so
  for (int c = c_lo; c < c_hi; ++c) {
    const int i = c - c_lo, st = i % STAGES;
    const int row0 = first_row + i * C, rows = min(end_row - row0, C);
    if (!dead && !mbar_wait(full + st, (i / STAGES) & 1)) dead = true;
    const float* Q = sm + st * stage_floats;
    const float* K = Q + C * DP;
    const float* PC = K + C * DP;
    const float* AT = PC + DP;
    const float* V = AT + C * C;
    float* mine = red + (size_t)(i & 1) * WD * C * VB;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      // r[t]: token half * 8 + (t ^ turn), so that what a lane keeps and what it hands on below are the same places of r
      // in every lane
      float r[8][2];
      const int turn = 2 * dgl;
#pragma unroll
      for (int t = 0; t < 8; ++t) {
        const Eight q = load8(Q + (half * 8 + (t & 1)) * DP + ((t ^ turn) & 6) * DP + d0);
        f32x2 a0 = mul2(q.p[0], S[0][0]), a1 = mul2(q.p[0], S[0][1]);
#pragma unroll
        for (int j = 1; j < 4; ++j) {
          a0 = fma2(q.p[j], S[j][0], a0);
          a1 = fma2(q.p[j], S[j][1], a1);
        }
        float x, y;
        unpack2(a0, x, y);
        r[t][0] = x + y;
        unpack2(a1, x, y);
        r[t][1] = x + y;
      }
      // the chunk's own tokens: every group of channels takes its share of the s
      for (int s = dg; s < C; s += 4 * WD) {
        const float2 v = *reinterpret_cast<const float2*>(V + s * VB + vl);
#pragma unroll
        for (int t = 0; t < 8; t += 2) {
          const float2 a = *reinterpret_cast<const float2*>(AT + s * C + half * 8 + (t ^ turn));
          r[t][0] = fmaf(a.x, v.x, r[t][0]);
          r[t][1] = fmaf(a.x, v.y, r[t][1]);
          r[t + 1][0] = fmaf(a.y, v.x, r[t + 1][0]);
          r[t + 1][1] = fmaf(a.y, v.y, r[t + 1][1]);
        }
      }
      // over the four lanes of a column pair: lane dgl ends with tokens 2 dgl and 2 dgl + 1
#pragma unroll
      for (int t = 0; t < 4; ++t)
#pragma unroll
        for (int k = 0; k < 2; ++k) r[t][k] += __shfl_xor_sync(0xffffffffu, r[t + 4][k], 16);
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int k = 0; k < 2; ++k) r[t][k] += __shfl_xor_sync(0xffffffffu, r[t + 2][k], 8);
#pragma unroll
      for (int t = 0; t < 2; ++t)
        *reinterpret_cast<float2*>(mine + ((size_t)wd * C + half * 8 + 2 * dgl + t) * VB + vl) = make_float2(r[t][0], r[t][1]);
    }
    {
      const Eight p = load8(PC + d0);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        S[j][0] = mul2(p.p[j], S[j][0]);
        S[j][1] = mul2(p.p[j], S[j][1]);
      }
    }
#pragma unroll
    for (int s = 0; s < C; ++s) {
      const Eight k = load8(K + s * DP + d0);
      const float2 v = *reinterpret_cast<const float2*>(V + s * VB + vl);
      const f32x2 va = pack2(v.x, v.x), vb = pack2(v.y, v.y);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        S[j][0] = fma2(k.p[j], va, S[j][0]);
        S[j][1] = fma2(k.p[j], vb, S[j][1]);
      }
    }
    __syncthreads();  // the stage is free and the partial sums are complete
    if (tid == 0 && c + STAGES < c_hi) issue(c + STAGES);
    for (int e = tid; e < rows * (VB / 2); e += blockDim.x) {
      const int t = e / (VB / 2), v = (e - t * (VB / 2)) * 2, gv = blockIdx.z * VB + v;
      float2 sum = *reinterpret_cast<const float2*>(mine + (size_t)t * VB + v);
      for (int k = 1; k < WD; ++k) {
        const float2 p = *reinterpret_cast<const float2*>(mine + ((size_t)k * C + t) * VB + v);
        sum.x += p.x;
        sum.y += p.y;
      }
      if (!FMS_IN(row0 + t, n_tokens)) continue;
      float* dst = o + (size_t)(row0 + t) * heads * vdim + (size_t)head * vdim + gv;
      if (vdim % 2 == 0) {
        if (gv < vdim) *reinterpret_cast<float2*>(dst) = sum;
      } else {
        if (gv < vdim) dst[0] = sum.x;
        if (gv + 1 < vdim) dst[1] = sum.y;
      }
    }
  }
  if (dead) {
    if (error_flag) atomicExch(error_flag, 4);
    for (int i = 0; i < STAGES; ++i)  // whatever is still on its way gets its time to arrive
      for (int ph = 0; ph < 2; ++ph) mbar_wait(full + i, ph);
  }
  if (write_state) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      if (v0 + i >= vdim) continue;
      float* p = state + (((size_t)slot * heads + head) * vdim + v0 + i) * dim;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int d = d0 + 2 * j;
        float x, y;
        unpack2(S[j][i], x, y);
        if (d < dim) p[d] = x;
        if (d + 1 < dim) p[d + 1] = y;
      }
    }
  }
}

// ---- a decode step ---------------------------------------------------------------------------------------
// L lanes hold a row of the state (a value column's dim key channels, 4 * N a lane); a warp takes 32 / L rows at once and
// ROWS such groups a tile.
constexpr int DECODE_WARPS = 8;

// sums r[0 .. COUNT) over the L lanes of a row by halves: a lane ends with the row whose number is returned, in r[0]
template <int COUNT, int L> __device__ __forceinline__ int rows_sum(float (&r)[COUNT], int lane) {
  int row = 0, half = COUNT;
#pragma unroll
  for (int o = L / 2; o > 0; o >>= 1) {
    if (half > 1) {
      half >>= 1;
      const bool hi = lane & o;
#pragma unroll
      for (int j = 0; j < COUNT / 2; ++j) {
        if (j < half) {
          const float other = __shfl_xor_sync(0xffffffffu, hi ? r[j] : r[j + half], o);
          r[j] = (hi ? r[j + half] : r[j]) + other;
        }
      }
      if (hi) row += half;
    } else {
      r[0] += __shfl_xor_sync(0xffffffffu, r[0], o);
    }
  }
  return row;
}

// proj: a row a sequence, [q: heads x dim | k | v: heads x vdim | ...], u at u_col, the gates' logits at gate_col;
// out [rows, heads * vdim] = o / sqrt(mean over the head(o^2) + eps) * norm[vdim] * silu(gate)
template <typename T, typename TW, int L, int N>
__global__ void __launch_bounds__(32 * DECODE_WARPS, 2) gla_decode_kernel(const T* proj, int stride, int u_col, int rank, const TW* w,
                                                                       const float* bias, double inv_tau, float q_scale, float* state,
                                                                       const int* slots, int gate_col, const float* norm, float eps, T* out,
                                                                       int heads, int dim, int vdim, int write_state, int n_slots) {
  constexpr int ROWS = N == 1 ? L / 2 : 8, PER = 32 / L;  // 16 rows a warp and tile (N == 2: 8)
  extern __shared__ __align__(16) float sm[];  // [rank]
  __shared__ __align__(16) float qs[256], ks[256], as[256];
  __shared__ float scratch[33];
  float* os = sm + ((rank + 3) & ~3);  // [vdim]
  float* vs = os + vdim;               // [vdim]
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int slot = __ldcg(slots + seq);
  if (!FMS_IN(slot, n_slots)) return;  // the whole block alike
  const T* row = proj + (size_t)seq * stride;
  float* st = state + ((size_t)slot * heads + head) * vdim * dim;
  const int sub = lane / L, at = (lane % L) * 4;  // the lane's row within a group and its first channel
  float4 S[ROWS][N];
  auto load = [&](int base) {
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
      const int v = base + j * PER + sub;
#pragma unroll
      for (int e = 0; e < N; ++e)
        S[j][e] = v < vdim && at + e * 4 * L < dim ? __ldcg(reinterpret_cast<const float4*>(st + (size_t)v * dim + at + e * 4 * L)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  load(warp * ROWS * PER);
  for (int r = tid; r < rank; r += blockDim.x) sm[r] = to_f32(row[u_col + r]);
  for (int d = tid; d < 256; d += blockDim.x) {
    qs[d] = d < dim ? to_f32(row[(size_t)head * dim + d]) * q_scale : 0.f;
    ks[d] = d < dim ? to_f32(row[(size_t)(heads + head) * dim + d]) : 0.f;
  }
  for (int v = tid; v < vdim; v += blockDim.x) vs[v] = to_f32(row[2 * (size_t)heads * dim + (size_t)head * vdim + v]);
  __syncthreads();
  for (int d = tid; d < 256; d += blockDim.x) {
    float a = 0.f;
    if (d < dim) {
      const TW* wr = w + ((size_t)head * dim + d) * rank;
      float z = bias[(size_t)head * dim + d], z2 = 0.f;
      int r = 0;
#pragma unroll 4
      for (; r + 1 < rank; r += 2) {
        z = fmaf(to_f32(wr[r]), sm[r], z);
        z2 = fmaf(to_f32(wr[r + 1]), sm[r + 1], z2);
      }
      if (r < rank) z = fmaf(to_f32(wr[r]), sm[r], z);
      // taken in double and rounded once: a decay's error compounds over a sequence
      const double m = -(double)(z + z2);
      a = (float)exp(-(m > 40.0 ? m : log1p(exp(m))) * inv_tau);
    }
    as[d] = a;
  }
  __syncthreads();
  float4 q[N], k[N], a[N];
#pragma unroll
  for (int e = 0; e < N; ++e) {
    q[e] = *reinterpret_cast<const float4*>(qs + at + e * 4 * L);
    k[e] = *reinterpret_cast<const float4*>(ks + at + e * 4 * L);
    a[e] = *reinterpret_cast<const float4*>(as + at + e * 4 * L);
  }
  for (int base = warp * ROWS * PER; base < vdim; base += DECODE_WARPS * ROWS * PER) {  // the whole warp alike
    if (base != warp * ROWS * PER) load(base);
    float r[ROWS];
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
      const int v = base + j * PER + sub;
      const float x = v < vdim ? vs[v] : 0.f;
      r[j] = 0.f;
#pragma unroll
      for (int e = 0; e < N; ++e) {
        float4 s = S[j][e];
        s.x = fmaf(a[e].x, s.x, k[e].x * x), s.y = fmaf(a[e].y, s.y, k[e].y * x);
        s.z = fmaf(a[e].z, s.z, k[e].z * x), s.w = fmaf(a[e].w, s.w, k[e].w * x);
        r[j] += fmaf(s.x, q[e].x, s.y * q[e].y) + fmaf(s.z, q[e].z, s.w * q[e].w);
        if (write_state && v < vdim && at + e * 4 * L < dim) *reinterpret_cast<float4*>(st + (size_t)v * dim + at + e * 4 * L) = s;
      }
    }
    const int mine = base + rows_sum<ROWS, L>(r, lane) * PER + sub;
    if (mine < vdim) os[mine] = r[0];  // lanes that end with the same row write the same sum
  }
  __syncthreads();
  float ss = 0.f;
  for (int v = tid; v < vdim; v += blockDim.x) ss = fmaf(os[v], os[v], ss);
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)vdim + eps);
  for (int v = tid; v < vdim; v += blockDim.x) {
    const float g = to_f32(row[gate_col + (size_t)head * vdim + v]);
    out[((size_t)seq * heads + head) * vdim + v] = from_f32<T>(os[v] * inv * norm[v] * (g / (1.f + expf(-g))));
  }
}

int padded_dim(int dim) { return dim <= 32 ? 32 : (dim <= 64 ? 64 : (dim <= 128 ? 128 : 256)); }
int value_run(int vdim) { return vdim > 16 ? 32 : 16; }  // value columns of a block
int padded_vdim(int vdim) { return (vdim + value_run(vdim) - 1) / value_run(vdim) * value_run(vdim); }
}  // namespace

FMS_API int fms_gla_chunk_tokens() { return C; }
// floats of one (chunk, head)'s record
FMS_API long fms_gla_record_floats(int dim, int vdim) {
  const long DP = padded_dim(dim);
  return 2L * C * DP + DP + C * C + (long)C * padded_vdim(vdim);
}

// proj: rows of `stride` values, [q: heads x dim | k: heads x dim | v: heads x vdim | ...], u at columns u_col .. u_col + rank;
// w [heads * dim, rank], bias float32 [heads * dim]; records: float32 scratch of n_chunks * heads records, 16-byte aligned;
// chunk_rows [n_chunks, 2], first_chunk [n_seqs + 1]: runs of fms_gla_chunk_tokens() rows of every sequence; state float32
// [slots, heads, vdim, dim]; o float32 [tokens, heads * vdim].
FMS_API int fms_gla_chunked(const void* proj, int dtype, int stride, int u_col, int rank, const void* w, int w_dtype,
                            const float* bias, float tau, float q_scale, const int* chunk_rows, const int* first_chunk, int n_chunks,
                            float* records, float* state, float* o, const int* slots, int n_tokens, int n_seqs, int heads, int dim,
                            int vdim, int write_state, int n_slots, int* error_flag, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0 || n_chunks <= 0) return 0;
  if (heads <= 0 || heads > 65535 || dim <= 0 || dim > 256 || vdim <= 0 || rank <= 0 || rank > 1024 || !(tau > 0.f))
    return fms_fail("gla_chunked: %d heads, dim %d (up to 256), vdim %d, rank %d (up to 1024), tau %f", heads, dim, vdim, rank, tau);
  if ((uintptr_t)records % 16 || (uintptr_t)o % 8) return fms_fail("gla_chunked: scratch and results must be aligned");
  const int DP = padded_dim(dim), VB = value_run(vdim), VP = padded_vdim(vdim);
  const size_t item = dtype == FMS_BF16 ? 2 : 4;
  const size_t prep = ((size_t)3 * C * DP + C * 4 + (size_t)C * ((rank + 3) & ~3)) * sizeof(float) +
                      (size_t)C * (2 * DP + ((vdim + 7) & ~7)) * item;
  // 16-byte copies: every row of a head's values starts on 16 bytes and its size is a multiple of them
  const bool rows16 = (uintptr_t)proj % 16 == 0 && (size_t)stride * item % 16 == 0;
  const int vec_qk = rows16 && (size_t)dim * item % 16 == 0;
  const int vec_v = rows16 && (size_t)vdim * item % 16 == 0 && (size_t)2 * heads * dim * item % 16 == 0;
  const size_t prep_smem = prep > 4 * C * C * sizeof(float) ? prep : 4 * C * C * sizeof(float);
  FMS_DISPATCH_DTYPE(dtype, T, FMS_DISPATCH_DTYPE(w_dtype, TW, {
    if (prep_smem > 48 * 1024)
      cudaFuncSetAttribute(gla_chunk_prepare_kernel<T, TW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)prep_smem);
    fms_launch(gla_chunk_prepare_kernel<T, TW>, dim3(n_chunks, heads), dim3(PREP_THREADS), prep_smem, stream, (const T*)proj, stride,
               u_col, rank, (const TW*)w, bias, (float)(1.0 / (double)tau), chunk_rows, records, heads, dim, vdim, DP, VP, VB, q_scale,
               n_tokens, vec_qk, vec_v);
  }));
  if (fms_launch_status("gla_chunk_prepare")) return 1;
#define FMS_GLA_SCAN(DP_, VB_)                                                                                              \
  do {                                                                                                                      \
    constexpr size_t smem = ((size_t)STAGES * (2 * C * DP_ + DP_ + C * C + C * VB_) + (size_t)2 * (DP_ / 32) * C * VB_) * sizeof(float); \
    static_assert(smem <= 220 * 1024, "stages and sums fit shared memory");                                                 \
    cudaFuncSetAttribute(gla_chunk_scan_kernel<DP_, VB_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(smem < 116 * 1024 ? 116 * 1024 : smem)); \
    /* up to a block a multiprocessor: as much shared memory as keeps a second one away */                                  \
    const size_t want = (long)n_seqs * heads * (VP / VB) <= 148 && smem < 116 * 1024 ? 116 * 1024 : smem;                    \
    fms_launch(gla_chunk_scan_kernel<DP_, VB_>, dim3(n_seqs, heads, VP / VB), dim3(DP_ / 32 * (VB_ / 16) * 32), want, stream, \
               (const float*)records, chunk_rows, first_chunk, state, o, slots, heads, dim, vdim, VP, write_state, n_slots,  \
               n_tokens, error_flag);                                                                                        \
  } while (0)
  if (VB == 32) {
    if (DP == 32) FMS_GLA_SCAN(32, 32); else if (DP == 64) FMS_GLA_SCAN(64, 32);
    else if (DP == 128) FMS_GLA_SCAN(128, 32); else FMS_GLA_SCAN(256, 32);
  } else {
    if (DP == 32) FMS_GLA_SCAN(32, 16); else if (DP == 64) FMS_GLA_SCAN(64, 16);
    else if (DP == 128) FMS_GLA_SCAN(128, 16); else FMS_GLA_SCAN(256, 16);
  }
#undef FMS_GLA_SCAN
  return fms_launch_status("gla_chunk_scan");
}

// One token of every sequence: row i of proj belongs to the sequence in slots[i].  norm [vdim] float32; out [n_seqs, heads * vdim]
// in proj's dtype.  dim a multiple of 4, state 16-byte aligned.
FMS_API int fms_gla_decode(const void* proj, int dtype, int stride, int u_col, int rank, const void* w, int w_dtype, const float* bias,
                           float tau, float q_scale, float* state, const int* slots, int gate_col, const float* norm, float eps, void* out,
                           int n_seqs, int heads, int dim, int vdim, int write_state, int n_slots, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (heads <= 0 || heads > 65535 || dim <= 0 || dim > 256 || dim % 4 || vdim <= 0 || vdim > 4096 || rank <= 0 || rank > 1024 || !(tau > 0.f) ||
      (uintptr_t)state % 16)
    return fms_fail("gla_decode: %d heads, dim %d (a multiple of 4 up to 256), vdim %d, rank %d (up to 1024), tau %f", heads, dim, vdim, rank, tau);
  const size_t smem = (size_t)(((rank + 3) & ~3) + 2 * vdim) * sizeof(float);
#define FMS_GLA_DECODE(L, N)                                                                                                \
  FMS_DISPATCH_DTYPE(dtype, T, FMS_DISPATCH_DTYPE(w_dtype, TW,                                                              \
                     fms_launch(gla_decode_kernel<T, TW, L, N>, dim3(n_seqs, heads), dim3(32 * DECODE_WARPS), smem, stream,  \
                                (const T*)proj, stride, u_col, rank, (const TW*)w, bias, 1.0 / (double)tau, q_scale, state,  \
                                slots, gate_col, norm, eps, (T*)out, heads, dim, vdim, write_state, n_slots)))
  if (dim <= 32) FMS_GLA_DECODE(8, 1);
  else if (dim <= 64) FMS_GLA_DECODE(16, 1);
  else if (dim <= 128) FMS_GLA_DECODE(32, 1);
  else FMS_GLA_DECODE(32, 2);
#undef FMS_GLA_DECODE
  return fms_launch_status("gla_decode");
}
