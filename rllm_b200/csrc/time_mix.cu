// What stands in front of a recurrence with token shift, float arithmetic throughout.
//
// shift_mix (a CTA takes one token, or a few in order): n = h / sqrt(mean(h^2) + eps) * w of the token's row and of the row before it in its
//   sequence (a portion's first token: the slot's `prev`, the normed row that the portion before ended with; no slot:
//   zeros), then `nmix` mixes n + (n_before - n) * mu_m, and optionally the plain row n and the same row under a
//   second norm's weight. The CTA of a portion's first token is the only one that touches its slot: having read
//   `prev` it writes the portion's last row there, which it norms itself, so that no CTA depends on another's order.
//   A row's norm is the same bits whichever CTA makes it. Without sequences (`token_seq` null) it is two norms of the
//   same rows in one pass.
// lowrank_decay: a = exp(-exp(W2 tanh(z) + b)) per column, z a row of `rank` numbers (the first projection's output). A thread
//   owns columns and walks the rank for eight tokens at a time, whose tanh(z) lie in shared memory; for steps of few
//   tokens eight lanes share a column and deal the rank out between them.
#include <initializer_list>
#include "common.cuh"
using namespace rllm;

namespace {

struct ShiftArgs {
  const float* h;                                    // [T, W]
  const float* w; const float* w2;                   // norm weights [W]; w2 null: no second norm
  float eps, eps2;
  const float* mu; int nmix;                         // [nmix, W]
  const int* token_seq; const int* cu_q; const int* state_slots;
  float* prev;                                       // [slots, W]
  void* mixes;                                       // [T, nmix, W]
  void* plain; void* second;                         // [T, W] or null
  int W;
};

template <typename TO, int VEC>
__device__ __forceinline__ void put(TO* p, const float (&v)[VEC]) {
  if constexpr (VEC == 1) {
    *p = from_f32<TO>(v[0]);
  } else if constexpr (sizeof(TO) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 u;
    u.x = *reinterpret_cast<unsigned*>(&a); u.y = *reinterpret_cast<unsigned*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
  }
}
template <int VEC>
__device__ __forceinline__ void get(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 1) v[0] = *p;
  else { const float4 t = *reinterpret_cast<const float4*>(p); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
}

// NV: pieces of VEC numbers a thread has of a row, held in registers (0: any number, the rows are read again). A CTA takes
// `per` tokens in order; what a token's norm gave serves the next one as the row before.
template <typename TO, int VEC, int NV>
__global__ void shift_mix_kernel(const ShiftArgs a, int T, int per) {
  pdl_launch();
  __shared__ float red[2][32];
  const int W = a.W, step = blockDim.x * VEC, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  constexpr int N = NV ? NV : 1;
  // the step's metadata and the norm's weight are written by no kernel of the step: read before the wait
  int t = blockIdx.x * per;
  const int t_end = min(T, t + per);
  int seq = -1, row0 = 0, row1 = 0, id = -1;
  auto find = [&](int at) {
    seq = a.token_seq[at]; row0 = a.cu_q[seq]; row1 = a.cu_q[seq + 1];
    id = a.state_slots ? a.state_slots[seq] : -1;
  };
  if (a.token_seq) find(t);
  float w[N][VEC];
  if (NV) {
#pragma unroll
    for (int q = 0; q < N; ++q) {
      const int i = threadIdx.x * VEC + q * step;
      if (i < W) get<VEC>(a.w + i, w[q]);
    }
  }
  pdl_wait();
  float x[N][VEC], o[N][VEC];                       // this token's row; the row before it, normed
  bool carried = false;                             // o holds the normed row of token t - 1
  for (; t < t_end; ++t) {
    if (a.token_seq && t >= row1) { find(t); carried = false; }
    const bool before = a.token_seq && t > row0;
    float* slot = a.token_seq && !before && id >= 0 ? a.prev + (size_t)id * W : nullptr;
    const float* hr = a.h + (size_t)t * W;
    // a second row is normed here: the one before (the CTA's first token), or the portion's last for its slot
    const float* other = before ? (carried ? nullptr : hr - W) : (slot && row1 - 1 > t ? a.h + (size_t)(row1 - 1) * W : nullptr);
    float y[N][VEC];
    float s0 = 0.f, s1 = 0.f;
    for (int q = 0; NV ? q < N : threadIdx.x * VEC + q * step < W; ++q) {
      const int i = threadIdx.x * VEC + q * step, r = NV ? q : 0;
      if (i >= W) break;
      get<VEC>(hr + i, x[r]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) s0 = fmaf(x[r][e], x[r][e], s0);
      if (other) {
        get<VEC>(other + i, y[r]);
#pragma unroll
        for (int e = 0; e < VEC; ++e) s1 = fmaf(y[r][e], y[r][e], s1);
      }
    }
    // both sums over the block in one go, each in the same order
    s0 = warp_sum(s0); s1 = warp_sum(s1);
    __syncthreads();
    if (lane == 0) { red[0][warp] = s0; red[1][warp] = s1; }
    __syncthreads();
    s0 = warp_sum(lane < nwarps ? red[0][lane] : 0.f) / (float)W;
    s1 = warp_sum(lane < nwarps ? red[1][lane] : 0.f) / (float)W;
    const float r = 1.f / sqrtf(s0 + a.eps), r2 = a.second ? 1.f / sqrtf(s0 + a.eps2) : 0.f, ro = 1.f / sqrtf(s1 + a.eps);
#pragma unroll
    for (int q = 0; NV ? q < N : threadIdx.x * VEC + q * step < W; ++q) {
      const int i = threadIdx.x * VEC + q * step, k = NV ? q : 0;
      if (i >= W) break;
      float n[VEC], p[VEC], z[VEC];
      if (!NV) {
        get<VEC>(hr + i, x[0]);
        get<VEC>(a.w + i, w[0]);
        if (other) get<VEC>(other + i, y[0]);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        n[e] = x[k][e] * r * w[k][e];
        if (other) y[k][e] = y[k][e] * ro * w[k][e];
        p[e] = 0.f;
      }
      if (before) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) p[e] = other ? y[k][e] : o[k][e];
      } else if (slot) {
        get<VEC>(slot + i, p);
        put<float, VEC>(slot + i, other ? y[k] : n);
      }
      for (int m = 0; m < a.nmix; ++m) {
        float mu[VEC];
        get<VEC>(a.mu + (size_t)m * W + i, mu);
#pragma unroll
        for (int e = 0; e < VEC; ++e) z[e] = fmaf(p[e] - n[e], mu[e], n[e]);
        put<TO, VEC>((TO*)a.mixes + ((size_t)t * a.nmix + m) * W + i, z);
      }
      if (a.plain) put<TO, VEC>((TO*)a.plain + (size_t)t * W + i, n);
      if (a.second) {
        float w2[VEC];
        get<VEC>(a.w2 + i, w2);
#pragma unroll
        for (int e = 0; e < VEC; ++e) z[e] = x[k][e] * r2 * w2[e];
        put<TO, VEC>((TO*)a.second + (size_t)t * W + i, z);
      }
      if (NV) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) o[k][e] = n[e];
      }
    }
    carried = NV > 0;
  }
}

constexpr int DT_TOKENS = 8, DT_MAX_RANK = 1024;

// eight numbers of a row of W2
template <typename TI>
__device__ __forceinline__ void get8(const TI* p, float (&w)[8]) {
  if constexpr (sizeof(TI) == 2) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(h2[e]); w[2 * e] = f.x; w[2 * e + 1] = f.y; }
  } else {
    const float4 u = *reinterpret_cast<const float4*>(p), v = *reinterpret_cast<const float4*>(p + 4);
    w[0] = u.x; w[1] = u.y; w[2] = u.z; w[3] = u.w; w[4] = v.x; w[5] = v.y; w[6] = v.z; w[7] = v.w;
  }
}
__device__ __forceinline__ void fma8(float w, const float* th, float (&acc)[DT_TOKENS]) {
  const float4 a = *reinterpret_cast<const float4*>(th), b = *reinterpret_cast<const float4*>(th + 4);
  acc[0] = fmaf(w, a.x, acc[0]); acc[1] = fmaf(w, a.y, acc[1]); acc[2] = fmaf(w, a.z, acc[2]); acc[3] = fmaf(w, a.w, acc[3]);
  acc[4] = fmaf(w, b.x, acc[4]); acc[5] = fmaf(w, b.y, acc[5]); acc[6] = fmaf(w, b.z, acc[6]); acc[7] = fmaf(w, b.w, acc[7]);
}

// Long portions, and sizes the other kernel does not take: CPT columns a thread (blockDim.x apart), the whole rank. VEC: W2's
// rows are read eight numbers at a time (rank a multiple of 8, rows on 16-byte boundaries).
template <typename TI, bool VEC, int CPT>
__global__ void lowrank_decay_kernel(const TI* __restrict__ z, long long ld, int rank, const TI* __restrict__ w2,
                                     const float* __restrict__ bias, float* __restrict__ out, int T, int C) {
  pdl_launch();
  pdl_wait();
  extern __shared__ __align__(16) float th[];         // [rank][DT_TOKENS]
  const int t0 = blockIdx.y * DT_TOKENS, n = min(DT_TOKENS, T - t0);
  for (int x = threadIdx.x; x < rank * DT_TOKENS; x += blockDim.x) {
    const int j = x % rank, tt = x / rank;
    th[j * DT_TOKENS + tt] = tt < n ? tanhf(to_f32(z[(long long)(t0 + tt) * ld + j])) : 0.f;
  }
  __syncthreads();
  const int c0 = blockIdx.x * blockDim.x * CPT + threadIdx.x;
  float acc[CPT][DT_TOKENS];
#pragma unroll
  for (int q = 0; q < CPT; ++q)
#pragma unroll
    for (int i = 0; i < DT_TOKENS; ++i) acc[q][i] = 0.f;
  const TI* wr[CPT];                                  // columns beyond C read the last one's row and store nothing
#pragma unroll
  for (int q = 0; q < CPT; ++q) wr[q] = w2 + (size_t)min(c0 + q * (int)blockDim.x, C - 1) * rank;
  if (VEC) {
    for (int j = 0; j < rank; j += 8) {
      float w[CPT][8];
#pragma unroll
      for (int q = 0; q < CPT; ++q) get8(wr[q] + j, w[q]);
#pragma unroll
      for (int e = 0; e < 8; ++e)
#pragma unroll
        for (int q = 0; q < CPT; ++q) fma8(w[q][e], th + (j + e) * DT_TOKENS, acc[q]);
    }
  } else {
    for (int j = 0; j < rank; ++j)
#pragma unroll
      for (int q = 0; q < CPT; ++q) fma8(to_f32(wr[q][j]), th + j * DT_TOKENS, acc[q]);
  }
#pragma unroll
  for (int q = 0; q < CPT; ++q) {
    const int c = c0 + q * (int)blockDim.x;
    if (c >= C) continue;
    const float b = bias[c];
#pragma unroll
    for (int i = 0; i < DT_TOKENS; ++i)
      if (i < n) out[(long long)(t0 + i) * C + c] = expf(-expf(acc[q][i] + b));
  }
}

// Steps of few tokens: eight neighbouring lanes share a column and eight numbers of every 64 of the rank each; their
// sums are joined by shuffles in lane order, after which each lane has one token's. The rows of W2, which no kernel
// writes, are asked for before the wait (the first 64 of the rank). The order of a sum depends on the rank alone.
template <typename TI>
__global__ void __launch_bounds__(256)
lowrank_decay_few_kernel(const TI* __restrict__ z, long long ld, int rank, const TI* __restrict__ w2,
                         const float* __restrict__ bias, float* __restrict__ out, int T, int C) {
  pdl_launch();
  extern __shared__ __align__(16) float th[];         // [rank][DT_TOKENS + 4]: lanes eight rows apart meet other banks
  constexpr int LD = DT_TOKENS + 4;
  const int part = threadIdx.x & 7, c = blockIdx.x * 32 + (threadIdx.x >> 3), cc = min(c, C - 1);
  const TI* wr = w2 + (size_t)cc * rank;
  float w[8];
  if (part * 8 < rank) get8(wr + part * 8, w);
  const float b = bias[cc];
  pdl_wait();
  const int t0 = blockIdx.y * DT_TOKENS, n = min(DT_TOKENS, T - t0);
  for (int x = threadIdx.x; x < rank * DT_TOKENS; x += blockDim.x) {
    const int j = x % rank, tt = x / rank;
    th[j * LD + tt] = tt < n ? tanhf(to_f32(z[(long long)(t0 + tt) * ld + j])) : 0.f;
  }
  __syncthreads();
  float acc[DT_TOKENS];
#pragma unroll
  for (int i = 0; i < DT_TOKENS; ++i) acc[i] = 0.f;
  for (int j = part * 8; j < rank; j += 64) {
    if (j >= 64) get8(wr + j, w);
#pragma unroll
    for (int e = 0; e < 8; ++e) fma8(w[e], th + (j + e) * LD, acc);
  }
#pragma unroll
  for (int i = 0; i < DT_TOKENS; ++i) {
    acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], 1);
    acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], 2);
    acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], 4);
  }
  float v = acc[0];
#pragma unroll
  for (int i = 1; i < DT_TOKENS; ++i) v = part == i ? acc[i] : v;
  if (c < C && part < n) out[(long long)(t0 + part) * C + c] = expf(-expf(v + b));
}

template <typename TO>
int launch_shift(const ShiftArgs& a, int T, bool vec, cudaStream_t s) {
  const int pieces = a.W / (vec ? 4 : 1);
  const int threads = pieces >= 1024 && vec ? 512 : pieces >= 256 ? 256 : pieces >= 128 ? 128 : 64;
  const int nv = (pieces + threads - 1) / threads;
  // long portions: four tokens a CTA share the norms of their rows and the shares (mu) in the L1 cache
  const int per = T >= 1024 ? 4 : 1;
  const dim3 grid((T + per - 1) / per), block(threads);
#define GO(V, NV) return launch_ex(shift_mix_kernel<TO, V, NV>, grid, block, 0, s, 1, a, T, per)
  if (!vec) GO(1, 0);
  if (nv == 1) GO(4, 1);
  if (nv == 2) GO(4, 2);
  if (nv <= 4) GO(4, 4);
  GO(4, 0);
#undef GO
}

}  // namespace

// h float [T, W]. mixes: [T, nmix, W] of type dt (nmix 0: none), mu float [nmix, W]. token_seq [T], cu_q [sequences + 1];
// state_slots [sequences] (-1 or null: no slot) into prev float [slots, W]. plain, second: [T, W] of type dt, or null.
RLLM_API int rllm_shift_mix(int dt, const float* h, const float* w, float eps, const float* w2, float eps2, const float* mu,
                            int nmix, const int* token_seq, const int* cu_q, const int* state_slots, float* prev,
                            void* mixes, void* plain, void* second, int T, int W, void* stream) {
  if (T <= 0) return 0;
  if (W <= 0 || nmix < 0 || (nmix && (!mu || !mixes)) || (second && !w2) || (token_seq && !cu_q) || (state_slots && !prev))
    return ERR_BAD_SIZE;
  const ShiftArgs a = {h, w, second ? w2 : nullptr, eps, eps2, mu, nmix, token_seq, cu_q, state_slots, prev, mixes, plain, second, W};
  bool vec = W % 4 == 0;
  for (const void* p : {(const void*)h, (const void*)w, (const void*)w2, (const void*)mu, (const void*)prev, (const void*)mixes,
                        (const void*)plain, (const void*)second})
    vec = vec && ((uintptr_t)p & 15) == 0;
  if (dt == DT_F32) return launch_shift<float>(a, T, vec, (cudaStream_t)stream);
  if (dt == DT_BF16) return launch_shift<bf16>(a, T, vec, (cudaStream_t)stream);
  return ERR_BAD_DTYPE;
}

// z: [T, >= rank] of type dt with row stride ld; w2 [C, rank] of type dt; bias float [C]; out float [T, C].
RLLM_API int rllm_lowrank_decay(int dt, const void* z, long long ld, int rank, const void* w2, const float* bias, float* out,
                                int T, int C, void* stream) {
  if (T <= 0 || C <= 0) return 0;
  if (rank <= 0 || rank > DT_MAX_RANK) return ERR_BAD_SIZE;
  const int row_tiles = (T + DT_TOKENS - 1) / DT_TOKENS;
  if (row_tiles > 65535) return ERR_TOO_LARGE;
  const bool vec = rank % 8 == 0 && !((uintptr_t)w2 & 15);
  cudaStream_t s = (cudaStream_t)stream;
  if (vec && row_tiles < 16) {
    const dim3 grid((C + 31) / 32, row_tiles);
    const size_t smem = (size_t)rank * (DT_TOKENS + 4) * sizeof(float);       // at most 48 KB
    if (dt == DT_F32)
      return launch_ex(lowrank_decay_few_kernel<float>, grid, dim3(256), smem, s, 1, (const float*)z, ld, rank, (const float*)w2, bias, out, T, C);
    if (dt == DT_BF16)
      return launch_ex(lowrank_decay_few_kernel<bf16>, grid, dim3(256), smem, s, 1, (const bf16*)z, ld, rank, (const bf16*)w2, bias, out, T, C);
    return ERR_BAD_DTYPE;
  }
  const int cpt = vec && C >= 512 ? 4 : 1;
  const dim3 grid((C + 128 * cpt - 1) / (128 * cpt), row_tiles);
  const size_t smem = (size_t)rank * DT_TOKENS * sizeof(float);
#define GO(TI, V, N) return launch_ex(lowrank_decay_kernel<TI, V, N>, grid, dim3(128), smem, s, 1, (const TI*)z, ld, rank, (const TI*)w2, bias, out, T, C)
  if (dt == DT_F32) { if (cpt == 4) GO(float, true, 4); if (vec) GO(float, true, 1); GO(float, false, 1); }
  if (dt == DT_BF16) { if (cpt == 4) GO(bf16, true, 4); if (vec) GO(bf16, true, 1); GO(bf16, false, 1); }
#undef GO
  return ERR_BAD_DTYPE;
}
