// Linear attention with a constant decay per head:  S_t = d_h S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t,  with q, k, v = silu of the raw
// projections (applied while they are loaded).  The state of a sequence lives in its slot in float and is carried from step to step.
//
// Token by token (lightning_scan_kernel): steps of single tokens, short portions, float32 serving and sizes off the tensor-core
// tiles.  A block owns up to 32 column groups of one (entry, head); the rows of a column group are dealt to the block's row groups,
// every thread keeps RPT x V cells of the state in registers, so a decoded token is one read and one write of the state with
// RPT wide loads in flight per thread; the partial read-outs of a token are added one token later, behind the next token's barrier.
//
// Chunks of 64 tokens (lightning_chunk_kernel): prompt portions over bf16 operands.  With i, j counted from the chunk's start:
//   o_i = d^(i+1) S^T q_i + sum_{j <= i} d^(i-j) (q_i . k_j) v_j        S' = d^n S + sum_j d^(n-1-j) k_j v_j^T
// as tensor-core products.  S stays in float registers (accumulator fragments); as an operand it is split into two bf16 terms
// (hi + lo, relative error 2^-17), and so are the decayed keys of the state update, so the state is never rounded to 16 bits.
// The powers of d come from a table formed in float64.  Compiled WITHOUT fast-math.
#include <cuda_bf16.h>

#include <cstdint>

#include "hybrid_kernels.h"

namespace {

constexpr int kChunk = NRL_LIGHTNING_CHUNK;
constexpr int kMinChunked = 16;          // entries with fewer tokens run token by token
constexpr int kMaxGroups = 32;           // column groups per block of the scan
__host__ __device__ constexpr int pre_of(int v) { return v == 4 ? 4 : 8; }      // q / k values a thread fetches ahead per token

__device__ __forceinline__ float silu_(float x) { return x / (1.f + expf(-x)); }

template <int V>
__device__ __forceinline__ void ldv(const float* p, float (&v)[V]) {
  if constexpr (V == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  } else {
    v[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void stv(float* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}

struct ScanArgs {
  const float* qkv;
  long sq;
  int col_q, col_k, col_v;
  const float* pows;
  int npow;
  float* state;
  float* o;
  const int* cu;
  const int* start;
  const int* state_slot;
  int heads, D, Dv;
  int max_tokens;      // > 0: entries with more tokens are left to the chunk kernel
};

// grid (entry, head, column slice); threads = CG column groups x RG row groups; thread (rg, cg): rows rg RPT .. rg RPT + RPT - 1 of V
// columns.  The next token's raw values are fetched while the current token is computed and pass through silu when they are staged.
template <int V, int RPT, int MAXT>
__global__ void __launch_bounds__(MAXT, 512 / MAXT) lightning_scan_kernel(const ScanArgs a, int CG, int RG) {
  constexpr int kPre = pre_of(V);
  extern __shared__ __align__(16) float sm[];
  const int e = blockIdx.x, h = blockIdx.y, D = a.D, Dv = a.Dv, DR = RG * RPT;
  const int t0 = a.cu[e], t1 = a.cu[e + 1];
  if (t0 >= t1 || (a.max_tokens > 0 && t1 - t0 > a.max_tokens)) return;
  float* stage = sm;                                       // [2][2 DR]: silu(q) | silu(k), zero behind D
  float* part = sm + 4 * DR;                               // [2][RG][CG * V]
  const int tid = threadIdx.x, nth = blockDim.x, cg = tid % CG, rg = tid / CG, base = blockIdx.z * CG * V, c = base + cg * V;
  const int cols = min(CG * V, Dv - base);
  const bool live = rg < RG && c < Dv;                     // V = 4 goes with Dv % 4 == 0: a group is whole or absent
  float* gS = a.state + (static_cast<long>(a.state_slot[e]) * a.heads + h) * D * Dv;
  const bool carried = a.start[e] > 0;
  float S[RPT][V];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = rg * RPT + i;
#pragma unroll
    for (int x = 0; x < V; ++x) S[i][x] = 0.f;
    if (live && carried && d < D) ldv<V>(gS + static_cast<long>(d) * Dv + c, S[i]);
  }
  if (DR != D) {
    for (int i = tid; i < 4 * DR; i += nth) stage[i] = 0.f;
    __syncthreads();
  }
  const float decay = a.pows[static_cast<long>(h) * a.npow + 1];
  float pre[kPre], pre_v[V];
  auto fetch = [&](int t) {
    const float* row = a.qkv + static_cast<long>(t) * a.sq;
#pragma unroll
    for (int i = 0; i < kPre; ++i) {
      const int idx = tid + i * nth;
      if (idx < 2 * D) pre[i] = idx < D ? row[a.col_q + h * D + idx] : row[a.col_k + h * D + idx - D];
    }
#pragma unroll
    for (int x = 0; x < V; ++x) pre_v[x] = live ? row[a.col_v + h * Dv + c + x] : 0.f;
  };
  auto emit = [&](int t) {                                 // the read-out of token t from its partial sums
    const float* p = part + (t & 1) * RG * CG * V;
    for (int x = tid; x < cols; x += nth) {
      float s = 0.f;
      for (int r = 0; r < RG; ++r) s += p[r * CG * V + x];
      a.o[static_cast<long>(t) * a.heads * Dv + h * Dv + base + x] = s;
    }
  };
  fetch(t0);
  for (int t = t0; t < t1; ++t) {
    float* qk = stage + (t & 1) * 2 * DR;
#pragma unroll
    for (int i = 0; i < kPre; ++i) {
      const int idx = tid + i * nth;
      if (idx < 2 * D) qk[idx < D ? idx : idx - D + DR] = silu_(pre[i]);
    }
    float v[V], acc[V];
#pragma unroll
    for (int x = 0; x < V; ++x) {
      v[x] = silu_(pre_v[x]);
      acc[x] = 0.f;
    }
    __syncthreads();
    if (t + 1 < t1) fetch(t + 1);
    if (t > t0) emit(t - 1);
    if (live) {
      const float4* q4 = reinterpret_cast<const float4*>(qk + rg * RPT);
      const float4* k4 = reinterpret_cast<const float4*>(qk + DR + rg * RPT);
#pragma unroll
      for (int i = 0; i < RPT / 4; ++i) {
        const float4 qa = q4[i], ka = k4[i];
        const float q[4] = {qa.x, qa.y, qa.z, qa.w}, k[4] = {ka.x, ka.y, ka.z, ka.w};
#pragma unroll
        for (int y = 0; y < 4; ++y)
#pragma unroll
          for (int x = 0; x < V; ++x) {
            float& cell = S[4 * i + y][x];
            cell = decay * cell + k[y] * v[x];
            acc[x] += cell * q[y];
          }
      }
      float* p = part + ((t & 1) * RG + rg) * CG * V + cg * V;
#pragma unroll
      for (int x = 0; x < V; ++x) p[x] = acc[x];
    }
  }
  __syncthreads();
  emit(t1 - 1);
  if (live) {
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg * RPT + i;
      if (d < D) stv<V>(gS + static_cast<long>(d) * Dv + c, S[i]);
    }
  }
}

// Any size: the state stays in global memory, thread per column.
__global__ void lightning_scan_global_kernel(const ScanArgs a) {
  const int e = blockIdx.x, h = blockIdx.y, D = a.D, Dv = a.Dv;
  const int t0 = a.cu[e], t1 = a.cu[e + 1];
  if (t0 >= t1 || (a.max_tokens > 0 && t1 - t0 > a.max_tokens)) return;
  float* gS = a.state + (static_cast<long>(a.state_slot[e]) * a.heads + h) * D * Dv;
  const bool carried = a.start[e] > 0;
  const float decay = a.pows[static_cast<long>(h) * a.npow + 1];
  for (int c = threadIdx.x; c < Dv; c += blockDim.x) {
    for (int t = t0; t < t1; ++t) {
      const float* row = a.qkv + static_cast<long>(t) * a.sq;
      const float v = silu_(row[a.col_v + h * Dv + c]);
      float acc = 0.f;
      for (int d = 0; d < D; ++d) {
        float* cell = gS + static_cast<long>(d) * Dv + c;
        const float s = decay * ((carried || t > t0) ? *cell : 0.f) + silu_(row[a.col_k + h * D + d]) * v;
        *cell = s;
        acc += s * silu_(row[a.col_q + h * D + d]);
      }
      a.o[static_cast<long>(t) * a.heads * Dv + h * Dv + c] = acc;
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------------
// chunks on the tensor cores
// ---------------------------------------------------------------------------------------------------------------------
constexpr int kThreads = 512;           // chunk kernel: 16 warps
constexpr int kPad = 8;                  // bf16 elements appended to a shared-memory row (ldmatrix without bank conflicts)

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ float2 unpack_bf16(uint32_t u) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u));
}
// x = hi + lo with both terms in bf16
__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  const float2 b = unpack_bf16(hi);
  lo = pack_bf16(x - b.x, y - b.y);
}
// silu of an operand that is rounded to bf16 next: exponential and division on the special-function unit
__device__ __forceinline__ float silu_fast(float x) {
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(e) : "f"(-1.4426950408889634f * x));
  return __fdividef(x, 1.f + fminf(e, 1e30f));             // the fast division wants a denominator below 2^126
}

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" :: "r"(dst), "l"(src));
}

// kChunk rows x WP columns (width real ones, rows from n on absent) of a raw projection.  A thread copies and later converts the
// same 16-byte pieces, so a piece needs no barrier between the two.
template <int WP>
__device__ __forceinline__ void fetch_tile(float* raw, const float* src, long sq, int n, int width) {
  constexpr int C4 = WP / 4;
#pragma unroll
  for (int it = 0; it < kChunk * C4 / kThreads; ++it) {
    const int idx = it * kThreads + threadIdx.x, r = idx / C4, c = (idx % C4) * 4;
    if (r < n && c < width) cp_async16(smem_u32(raw + idx * 4), src + static_cast<long>(r) * sq + c);
  }
}
// silu, rounded to bf16; absent pieces are zero
template <int WP>
__device__ __forceinline__ void convert_tile(__nv_bfloat16* dst, const float* raw, int n, int width) {
  constexpr int C4 = WP / 4, LD = WP + kPad;
#pragma unroll
  for (int it = 0; it < kChunk * C4 / kThreads; ++it) {
    const int idx = it * kThreads + threadIdx.x, r = idx / C4, c = (idx % C4) * 4;
    uint2 v = make_uint2(0u, 0u);
    if (r < n && c < width) {
      const float4 x = *reinterpret_cast<const float4*>(raw + idx * 4);
      v = make_uint2(pack_bf16(silu_fast(x.x), silu_fast(x.y)), pack_bf16(silu_fast(x.z), silu_fast(x.w)));
    }
    *reinterpret_cast<uint2*>(dst + r * LD + c) = v;
  }
}

// grid (entry, head); 16 warps.  For the chunk's output a warp owns 16 rows and NH groups of 16 value columns (four row tiles x four
// column parts; the row tile is rotated over the SM's four schedulers, since later rows see more keys), for the state [D, Dv] 16 rows
// and NU column groups (sizes that give fewer parts than warps leave warps idle).  The raw projections of the next chunk are copied to
// shared memory while the current one is computed.
template <int KS, int NV>      // padded D = 16 KS, padded Dv = 16 NV
__global__ void __launch_bounds__(kThreads, 1) lightning_chunk_kernel(const ScanArgs a) {
  constexpr int DP = 16 * KS, SW = 16 * NV, LDK = DP + kPad, LDV = SW + kPad;
  constexpr int NH = NV >= 4 ? NV / 4 : 1, NU = NV * KS >= 16 ? NV * KS / 16 : 1;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  float* rQ = reinterpret_cast<float*>(smem_raw);                             // [kChunk][DP] raw projections of the next chunk
  float* rK = rQ + kChunk * DP;                                               // [kChunk][DP]
  float* rV = rK + kChunk * DP;                                               // [kChunk][SW]
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(rV + kChunk * SW);     // [kChunk][LDK]
  __nv_bfloat16* sK = sQ + kChunk * LDK;                                      // [kChunk][LDK]
  __nv_bfloat16* sV = sK + kChunk * LDK;                                      // [kChunk][LDV]
  __nv_bfloat16* sH = sV + kChunk * LDV;                                      // [DP][LDV]: the state's leading terms
  __nv_bfloat16* sL = sH + DP * LDV;                                          // [DP][LDV]: the rest
  __shared__ float pw[kChunk + 1];
  const int e = blockIdx.x, h = blockIdx.y, D = a.D, Dv = a.Dv;
  const int t0 = a.cu[e], t1 = a.cu[e + 1];
  if (t1 - t0 < kMinChunked) return;
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, gq = lane >> 2, tq = lane & 3, mi = lane >> 3;
  const int rt = (w + (w >> 2)) & 3, nv0 = (w >> 2) * NH;
  const bool reader = nv0 < NV;
  auto fetch = [&](int t) {
    const int n = min(kChunk, t1 - t);
    const float* row = a.qkv + static_cast<long>(t) * a.sq;
    fetch_tile<DP>(rQ, row + a.col_q + h * D, a.sq, n, D);
    fetch_tile<DP>(rK, row + a.col_k + h * D, a.sq, n, D);
    fetch_tile<SW>(rV, row + a.col_v + h * Dv, a.sq, n, Dv);
    asm volatile("cp.async.commit_group;\n" ::);
  };
  fetch(t0);
  for (int i = threadIdx.x; i <= kChunk; i += kThreads) pw[i] = a.pows[static_cast<long>(h) * a.npow + i];
  const int m0 = (w % KS) * 16, u0 = (w / KS) * NU;        // the warp's part of the state: rows m0 .. m0 + 15, column groups u0 .. u0 + NU - 1
  const bool owner = u0 < NV;
  float* gS = a.state + (static_cast<long>(a.state_slot[e]) * a.heads + h) * D * Dv;
  const bool carried = a.start[e] > 0;
  float S[2 * NU][4];
#pragma unroll
  for (int i = 0; i < 2 * NU; ++i)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int d = m0 + gq + hf * 8, c = u0 * 16 + i * 8 + 2 * tq;
      float2 x = make_float2(0.f, 0.f);
      if (owner && carried && d < D && c < Dv) x = *reinterpret_cast<const float2*>(gS + static_cast<long>(d) * Dv + c);
      S[i][2 * hf] = x.x;
      S[i][2 * hf + 1] = x.y;
    }
  const int krow = (mi >> 1) * 8 + (lane & 7), kcol = (mi & 1) * 8, vrow = (mi & 1) * 8 + (lane & 7), vcol = (mi >> 1) * 8;
  for (int t = t0; t < t1; t += kChunk) {
    const int n = min(kChunk, t1 - t);
    asm volatile("cp.async.wait_group 0;\n" ::);
    convert_tile<DP>(sQ, rQ, n, D);
    convert_tile<DP>(sK, rK, n, D);
    convert_tile<SW>(sV, rV, n, Dv);
    if (t + kChunk < t1) fetch(t + kChunk);                // into this thread's own pieces, which it has just read
    if (owner) {
#pragma unroll
      for (int i = 0; i < 2 * NU; ++i)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          uint32_t hi, lo;
          split_bf16(S[i][2 * hf], S[i][2 * hf + 1], hi, lo);
          const int at = (m0 + gq + hf * 8) * LDV + u0 * 16 + i * 8 + 2 * tq;
          *reinterpret_cast<uint32_t*>(sH + at) = hi;
          *reinterpret_cast<uint32_t*>(sL + at) = lo;
        }
    }
    __syncthreads();
    if (reader && rt * 16 < n) {
      // ---- scores of the warp's rows against the chunk's keys up to the diagonal, and the read-out of the carried state ----
      float s[kChunk / 8][4], o[2 * NH][4];
#pragma unroll
      for (int i = 0; i < kChunk / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
      for (int i = 0; i < 2 * NH; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        uint32_t qf[4], b[4];
        ldsm_x4(smem_u32(sQ + (rt * 16 + vrow) * LDK + ks * 16 + vcol), qf);
#pragma unroll
        for (int np = 0; np < kChunk / 16; ++np) {
          if (np <= rt) {
            ldsm_x4(smem_u32(sK + (np * 16 + krow) * LDK + ks * 16 + kcol), b);
            mma_bf16(s[2 * np], qf, b[0], b[1]);
            mma_bf16(s[2 * np + 1], qf, b[2], b[3]);
          }
        }
#pragma unroll
        for (int nv = 0; nv < NH; ++nv) {
          ldsm_x4_t(smem_u32(sH + (ks * 16 + vrow) * LDV + (nv0 + nv) * 16 + vcol), b);
          mma_bf16(o[2 * nv], qf, b[0], b[1]);
          mma_bf16(o[2 * nv + 1], qf, b[2], b[3]);
          ldsm_x4_t(smem_u32(sL + (ks * 16 + vrow) * LDV + (nv0 + nv) * 16 + vcol), b);
          mma_bf16(o[2 * nv], qf, b[0], b[1]);
          mma_bf16(o[2 * nv + 1], qf, b[2], b[3]);
        }
      }
      const int i0 = rt * 16 + gq;
      const float f0 = pw[i0 + 1], f1 = pw[i0 + 9];
#pragma unroll
      for (int i = 0; i < 2 * NH; ++i) {
        o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1;
      }
#pragma unroll
      for (int kk = 0; kk < kChunk / 16; ++kk) {
        if (kk > rt) continue;
        uint32_t pa[4];
#pragma unroll
        for (int x = 0; x < 2; ++x) {                        // decay and causal mask in float
          const int j = kk * 16 + x * 8 + 2 * tq;
          float* sx = s[2 * kk + x];
          const float p0 = j <= i0 ? sx[0] * pw[i0 - j] : 0.f, p1 = j + 1 <= i0 ? sx[1] * pw[i0 - j - 1] : 0.f;
          const float p2 = j <= i0 + 8 ? sx[2] * pw[i0 + 8 - j] : 0.f, p3 = j + 1 <= i0 + 8 ? sx[3] * pw[i0 + 7 - j] : 0.f;
          pa[2 * x] = pack_bf16(p0, p1);
          pa[2 * x + 1] = pack_bf16(p2, p3);
        }
#pragma unroll
        for (int nv = 0; nv < NH; ++nv) {
          uint32_t b[4];
          ldsm_x4_t(smem_u32(sV + (kk * 16 + vrow) * LDV + (nv0 + nv) * 16 + vcol), b);
          mma_bf16(o[2 * nv], pa, b[0], b[1]);
          mma_bf16(o[2 * nv + 1], pa, b[2], b[3]);
        }
      }
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        if (i0 + 8 * hf >= n) continue;
        float* dst = a.o + static_cast<long>(t + i0 + 8 * hf) * a.heads * Dv + h * Dv;
#pragma unroll
        for (int i = 0; i < 2 * NH; ++i) {
          const int c = nv0 * 16 + i * 8 + 2 * tq;
          if (c < Dv) *reinterpret_cast<float2*>(dst + c) = make_float2(o[i][2 * hf], o[i][2 * hf + 1]);
        }
      }
    }
    if (owner) {
      // ---- S <- d^n S + sum_j d^(n-1-j) k_j v_j^T ----
      const float fn = pw[n];
#pragma unroll
      for (int i = 0; i < 2 * NU; ++i) {
        S[i][0] *= fn; S[i][1] *= fn; S[i][2] *= fn; S[i][3] *= fn;
      }
#pragma unroll
      for (int kk = 0; kk < kChunk / 16; ++kk) {
        if (kk * 16 >= n) break;
        float wj[4];                                         // decays of the tokens this thread's fragment columns stand for
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int j = kk * 16 + 2 * tq + (x & 1) + (x >> 1) * 8;
          wj[x] = j < n ? pw[n - 1 - j] : 0.f;
        }
        uint32_t kt[4], hi[4], lo[4];                        // K^T: rows = key channels, columns = tokens
        ldsm_x4_t(smem_u32(sK + (kk * 16 + krow) * LDK + m0 + kcol), kt);
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float2 kf = unpack_bf16(kt[x]);
          split_bf16(kf.x * wj[2 * (x >> 1)], kf.y * wj[2 * (x >> 1) + 1], hi[x], lo[x]);
        }
#pragma unroll
        for (int nv = 0; nv < NU; ++nv) {
          uint32_t b[4];
          ldsm_x4_t(smem_u32(sV + (kk * 16 + vrow) * LDV + (u0 + nv) * 16 + vcol), b);
          mma_bf16(S[2 * nv], hi, b[0], b[1]);
          mma_bf16(S[2 * nv + 1], hi, b[2], b[3]);
          mma_bf16(S[2 * nv], lo, b[0], b[1]);
          mma_bf16(S[2 * nv + 1], lo, b[2], b[3]);
        }
      }
    }
    __syncthreads();                                         // the tiles may be filled again
  }
  if (owner) {
#pragma unroll
    for (int i = 0; i < 2 * NU; ++i)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int d = m0 + gq + hf * 8, c = u0 * 16 + i * 8 + 2 * tq;
        if (d < D && c < Dv) *reinterpret_cast<float2*>(gS + static_cast<long>(d) * Dv + c) = make_float2(S[i][2 * hf], S[i][2 * hf + 1]);
      }
  }
}

template <int KS, int NV>
cudaError_t launch_chunk(const ScanArgs& a, int E, cudaStream_t s) {
  constexpr int DP = 16 * KS, SW = 16 * NV;
  constexpr size_t smem = sizeof(float) * kChunk * (2 * DP + SW) +
                          sizeof(__nv_bfloat16) * (2 * kChunk * (DP + kPad) + kChunk * (SW + kPad) + 2 * DP * (SW + kPad));
  auto kern = lightning_chunk_kernel<KS, NV>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return e;
    configured = true;
  }
  kern<<<dim3(E, a.heads), kThreads, smem, s>>>(a);
  return cudaGetLastError();
}

cudaError_t run_chunk(const ScanArgs& a, int E, cudaStream_t s) {
  if (!nrl_lightning_chunk_fits(a.D, a.Dv, a.npow) || a.sq % 4 != 0 || a.col_q % 4 != 0 || a.col_k % 4 != 0 || a.col_v % 4 != 0 ||
      reinterpret_cast<uintptr_t>(a.qkv) % 16 != 0 || reinterpret_cast<uintptr_t>(a.state) % 8 != 0 || reinterpret_cast<uintptr_t>(a.o) % 8 != 0)
    return cudaErrorInvalidValue;
  const int ks = a.D <= 32 ? 2 : a.D <= 64 ? 4 : 8, nv = a.Dv <= 32 ? 2 : a.Dv <= 64 ? 4 : 8;
#define NRL_LC(KS_, NV_) \
  if (ks == KS_ && nv == NV_) return launch_chunk<KS_, NV_>(a, E, s);
  NRL_LC(2, 2) NRL_LC(2, 4) NRL_LC(2, 8) NRL_LC(4, 2) NRL_LC(4, 4) NRL_LC(4, 8) NRL_LC(8, 2) NRL_LC(8, 4) NRL_LC(8, 8)
#undef NRL_LC
  return cudaErrorInvalidValue;
}

template <int V, int RPT, int MAXT>
cudaError_t launch_scan(const ScanArgs& a, int E, int CG, int RG, int slices, cudaStream_t s) {
  const int threads = (CG * RG + 31) / 32 * 32;
  const size_t smem = sizeof(float) * (4 * static_cast<size_t>(RG) * RPT + 2 * static_cast<size_t>(RG) * CG * V);
  lightning_scan_kernel<V, RPT, MAXT><<<dim3(E, a.heads, slices), threads, smem, s>>>(a, CG, RG);
  return cudaGetLastError();
}

// registers: V columns x RPT rows per thread; false when no layout fits
template <int V>
bool try_scan(const ScanArgs& a, int E, cudaStream_t s, cudaError_t* err) {
  const int groups = (a.Dv + V - 1) / V, CG = groups < kMaxGroups ? groups : kMaxGroups, slices = (groups + CG - 1) / CG;
  for (int cap = 256; cap <= 512; cap *= 2)
    for (int rpt = 4; rpt <= (V == 4 ? 16 : 32); rpt *= 2) {
      const int RG = (a.D + rpt - 1) / rpt, threads = (CG * RG + 31) / 32 * 32;
      if (threads > cap || 2 * a.D > pre_of(V) * threads) continue;
      const size_t smem = sizeof(float) * (4 * static_cast<size_t>(RG) * rpt + 2 * static_cast<size_t>(RG) * CG * V);
      if (smem > 48 * 1024) continue;
#define NRL_LS(RPT_) \
  if (rpt == RPT_) { \
    *err = threads <= 256 ? launch_scan<V, RPT_, 256>(a, E, CG, RG, slices, s) : launch_scan<V, RPT_, 512>(a, E, CG, RG, slices, s); \
    return true; \
  }
      NRL_LS(4) NRL_LS(8) NRL_LS(16)
      if constexpr (V == 1) NRL_LS(32)
#undef NRL_LS
    }
  return false;
}

cudaError_t run_scan(const ScanArgs& a, int E, int impl, cudaStream_t s) {
  cudaError_t err = cudaSuccess;
  if (impl != 2) {
    if (a.Dv % 4 == 0 && reinterpret_cast<uintptr_t>(a.state) % 16 == 0 && try_scan<4>(a, E, s, &err)) return err;
    if (try_scan<1>(a, E, s, &err)) return err;
    if (impl == 1) return cudaErrorInvalidValue;
  }
  const int th = a.Dv >= 256 ? 256 : (a.Dv + 31) / 32 * 32;
  lightning_scan_global_kernel<<<dim3(E, a.heads), th, 0, s>>>(a);
  return cudaGetLastError();
}

}  // namespace

extern "C" {

int nrl_lightning_chunk_fits(int D, int Dv, int npow) { return D % 8 == 0 && Dv % 8 == 0 && D >= 8 && Dv >= 8 && D <= 128 && Dv <= 128 && npow > kChunk; }

cudaError_t nrl_lightning_chunk(const float* qkv, long sq, int col_q, int col_k, int col_v, const float* pows, int npow, float* state, float* o,
                                const int* cu, const int* start, const int* state_slot, int E, int heads, int D, int Dv, cudaStream_t s) {
  const ScanArgs a = {qkv, sq, col_q, col_k, col_v, pows, npow, state, o, cu, start, state_slot, heads, D, Dv, 0};
  return E <= 0 ? cudaSuccess : run_chunk(a, E, s);
}

cudaError_t nrl_lightning_scan(const float* qkv, long sq, int col_q, int col_k, int col_v, const float* pows, int npow, float* state, float* o,
                               const int* cu, const int* start, const int* state_slot, int E, int heads, int D, int Dv, int single_token,
                               int chunk_ok, int impl, cudaStream_t s) {
  if (E <= 0) return cudaSuccess;
  if (D < 1 || Dv < 1 || heads < 1 || npow < 2 || impl < 0 || impl > 3) return cudaErrorInvalidValue;
  ScanArgs a = {qkv, sq, col_q, col_k, col_v, pows, npow, state, o, cu, start, state_slot, heads, D, Dv, 0};
  const bool fits = nrl_lightning_chunk_fits(D, Dv, npow) && sq % 4 == 0 && col_q % 4 == 0 && col_k % 4 == 0 && col_v % 4 == 0 &&
                    reinterpret_cast<uintptr_t>(qkv) % 16 == 0 && reinterpret_cast<uintptr_t>(state) % 8 == 0;
  if (impl == 3 && !fits) return cudaErrorInvalidValue;
  if (impl == 3 || (impl == 0 && chunk_ok && fits && !single_token)) {
    // long portions in chunks; entries of few tokens in the same step are left to the scan
    const cudaError_t e = run_chunk(a, E, s);
    if (e != cudaSuccess) return e;
    a.max_tokens = kMinChunked - 1;
    impl = 0;
  }
  return run_scan(a, E, impl, s);
}

}  // extern "C"
