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
//   owns columns and walks the rank for some tokens at a time, whose tanh(z) lie in shared memory; for steps of few
//   tokens the warps of a CTA deal the rank out between them. W2 is kept transposed, so that a warp reads runs of it.
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
// `per` tokens in order, the next one's row asked for before this one's sum; what a token's norm gave serves the next one
// as the row before.
// NMIX: the number of mixes where it is known when compiled; their shares, and the second norm's weight, then also stay
// in registers (0: any number, read where they are used). SHIFT false: no sequences, every row by itself.
template <typename TO, int VEC, int NV, int NMIX, bool SHIFT>
__global__ void __launch_bounds__(512, NV == 1 ? 2 : 1) shift_mix_kernel(const ShiftArgs a, int T, int per) {
  pdl_launch();
  __shared__ float red[2][32];
  const int W = a.W, step = blockDim.x * VEC, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  constexpr int N = NV ? NV : 1;
  constexpr bool KEPT = NV && (NMIX || !SHIFT);     // the second norm's weight stays in registers
  // the step's metadata and the norm's weight are written by no kernel of the step: read before the wait
  int t = blockIdx.x * per;
  const int t_end = min(T, t + per);
  int seq = -1, row0 = 0, row1 = 0, id = -1;
  auto find = [&](int at) {
    seq = a.token_seq[at]; row0 = a.cu_q[seq]; row1 = a.cu_q[seq + 1];
    id = a.state_slots ? a.state_slots[seq] : -1;
  };
  const bool shift = SHIFT && a.token_seq != nullptr;
  if (shift) find(t);
  float w[N][VEC], mus[NMIX ? NMIX : 1][N][VEC], w2[N][VEC];
  if (NV) {
#pragma unroll
    for (int q = 0; q < N; ++q) {
      const int i = threadIdx.x * VEC + q * step;
      if (i >= W) continue;
      get<VEC>(a.w + i, w[q]);
      if (NMIX) {
#pragma unroll
        for (int m = 0; m < NMIX; ++m) get<VEC>(a.mu + (size_t)m * W + i, mus[m][q]);
      }
      if (KEPT && a.second) get<VEC>(a.w2 + i, w2[q]);
    }
  }
  pdl_wait();
  float x[N][VEC], ahead[N][VEC], o[N][VEC];        // this token's row, the next one's; the row before it, normed
  auto ask = [&](int at) {
#pragma unroll
    for (int q = 0; q < N; ++q) {
      const int i = threadIdx.x * VEC + q * step;
      if (i < W) get<VEC>(a.h + (size_t)at * W + i, ahead[q]);
    }
  };
  if (NV && t < t_end) ask(t);
  bool carried = false;                             // o holds the normed row of token t - 1
  for (; t < t_end; ++t) {
    if (shift && t >= row1) { find(t); carried = false; }
    const bool before = shift && t > row0;
    float* slot = shift && !before && id >= 0 ? a.prev + (size_t)id * W : nullptr;
    const float* hr = a.h + (size_t)t * W;
    // a second row is normed here: the one before (the CTA's first token), or the portion's last for its slot
    const float* other = before ? (carried ? nullptr : hr - W) : (slot && row1 - 1 > t ? a.h + (size_t)(row1 - 1) * W : nullptr);
    float y[N][VEC], held[N][VEC];
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int q = 0; NV ? q < N : threadIdx.x * VEC + q * step < W; ++q) {
      const int i = threadIdx.x * VEC + q * step, r = NV ? q : 0;
      if (i >= W) break;
      if (NV) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[r][e] = ahead[r][e];
      } else {
        get<VEC>(hr + i, x[r]);
      }
      if (NV && slot) get<VEC>(slot + i, held[r]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) s0 = fmaf(x[r][e], x[r][e], s0);
      if (other) {
        get<VEC>(other + i, y[r]);
#pragma unroll
        for (int e = 0; e < VEC; ++e) s1 = fmaf(y[r][e], y[r][e], s1);
      }
    }
    if (NV && t + 1 < t_end) ask(t + 1);
    // both sums over the block in one go, each in the same order
    s0 = warp_sum(s0);
    if (other) s1 = warp_sum(s1);
    __syncthreads();
    if (lane == 0) { red[0][warp] = s0; red[1][warp] = s1; }
    __syncthreads();
    s0 = warp_sum(lane < nwarps ? red[0][lane] : 0.f) / (float)W;
    if (other) s1 = warp_sum(lane < nwarps ? red[1][lane] : 0.f) / (float)W;
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
        if (NV) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) p[e] = held[k][e];
        } else {
          get<VEC>(slot + i, p);
        }
        put<float, VEC>(slot + i, other ? y[k] : n);
      }
      if (NMIX) {
#pragma unroll
        for (int m = 0; m < NMIX; ++m) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) z[e] = fmaf(p[e] - n[e], mus[m][k][e], n[e]);
          put<TO, VEC>((TO*)a.mixes + ((size_t)t * NMIX + m) * W + i, z);
        }
      } else {
        for (int m = 0; m < a.nmix; ++m) {
          float mu[VEC];
          get<VEC>(a.mu + (size_t)m * W + i, mu);
#pragma unroll
          for (int e = 0; e < VEC; ++e) z[e] = fmaf(p[e] - n[e], mu[e], n[e]);
          put<TO, VEC>((TO*)a.mixes + ((size_t)t * a.nmix + m) * W + i, z);
        }
      }
      if (a.plain) put<TO, VEC>((TO*)a.plain + (size_t)t * W + i, n);
      if (a.second) {
        if (!KEPT) get<VEC>(a.w2 + i, w2[k]);
#pragma unroll
        for (int e = 0; e < VEC; ++e) z[e] = x[k][e] * r2 * w2[k][e];
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

// CPT neighbouring numbers of a row of W2^T
template <typename TI, int CPT>
__device__ __forceinline__ void get_cols(const TI* p, float (&w)[CPT]) {
  if constexpr (CPT == 4 && sizeof(TI) == 2) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    w[0] = a.x; w[1] = a.y; w[2] = b.x; w[3] = b.y;
  } else if constexpr (CPT == 4) {
    const float4 u = *reinterpret_cast<const float4*>(p);
    w[0] = u.x; w[1] = u.y; w[2] = u.z; w[3] = u.w;
  } else {
#pragma unroll
    for (int q = 0; q < CPT; ++q) w[q] = to_f32(p[q]);
  }
}
template <int N>
__device__ __forceinline__ void get_tokens(const float* th, float (&v)[N]) {
#pragma unroll
  for (int i = 0; i < N; i += 4) {
    const float4 a = *reinterpret_cast<const float4*>(th + i);
    v[i] = a.x; v[i + 1] = a.y; v[i + 2] = a.z; v[i + 3] = a.w;
  }
}
// tanh of a tile's rows, [rank][TT] in shared memory (zeros for the rows beyond n)
template <typename TI, int TT>
__device__ __forceinline__ void stage_tanh(float* th, const TI* z, long long ld, int rank, int n) {
  for (int x = threadIdx.x; x < rank * TT; x += blockDim.x) {
    const int j = x % rank, tt = x / rank;
    th[j * TT + tt] = tt < n ? tanhf(to_f32(z[tt * ld + j])) : 0.f;
  }
}

// Long portions: a thread owns CPT neighbouring columns and walks the whole rank for TT tokens.
template <typename TI, int CPT, int TT>
__global__ void __launch_bounds__(128)
lowrank_decay_kernel(const TI* __restrict__ z, long long ld, int rank, const TI* __restrict__ w2t,
                     const float* __restrict__ bias, float* __restrict__ out, int T, int C) {
  pdl_launch();
  pdl_wait();
  extern __shared__ __align__(16) float th[];         // [rank][TT]
  const int t0 = blockIdx.y * TT, n = min(TT, T - t0);
  stage_tanh<TI, TT>(th, z + (long long)t0 * ld, ld, rank, n);
  __syncthreads();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * CPT;       // C is a multiple of CPT
  if (c >= C) return;
  float acc[CPT][TT];
#pragma unroll
  for (int q = 0; q < CPT; ++q)
#pragma unroll
    for (int i = 0; i < TT; ++i) acc[q][i] = 0.f;
  const TI* wp = w2t + c;
#pragma unroll 4
  for (int j = 0; j < rank; ++j) {
    float w[CPT], v[TT];
    get_cols<TI, CPT>(wp + (size_t)j * C, w);
    get_tokens<TT>(th + j * TT, v);
#pragma unroll
    for (int q = 0; q < CPT; ++q)
#pragma unroll
      for (int i = 0; i < TT; ++i) acc[q][i] = fmaf(w[q], v[i], acc[q][i]);
  }
  float b[CPT];
#pragma unroll
  for (int q = 0; q < CPT; ++q) b[q] = bias[c + q];
#pragma unroll
  for (int i = 0; i < TT; ++i) {
    if (i >= n) break;
    float* o = out + (long long)(t0 + i) * C + c;
    float e[CPT];
#pragma unroll
    for (int q = 0; q < CPT; ++q) e[q] = expf(-expf(acc[q][i] + b[q]));
    if constexpr (CPT == 4) *reinterpret_cast<float4*>(o) = make_float4(e[0], e[1], e[2], e[3]);
    else
#pragma unroll
      for (int q = 0; q < CPT; ++q) o[q] = e[q];
  }
}

// Steps of few tokens: a CTA has 32 * CPT columns and eight tokens; its eight warps take every eighth number of the
// rank, and their sums meet in shared memory in warp order. A warp's first numbers of W2, which no kernel writes, are
// asked for before the wait. The order of a sum depends on the rank alone.
constexpr int DT_AHEAD = 8;
template <typename TI, int CPT>
__global__ void __launch_bounds__(256)
lowrank_decay_few_kernel(const TI* __restrict__ z, long long ld, int rank, const TI* __restrict__ w2t,
                         const float* __restrict__ bias, float* __restrict__ out, int T, int C) {
  pdl_launch();
  constexpr int TT = DT_TOKENS, COLS = 32 * CPT;
  extern __shared__ __align__(16) float th[];         // [rank][TT], then the sums [8][TT][COLS]
  float* sums = th + rank * TT;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = (blockIdx.x * 32 + lane) * CPT, cc = min(c, C - CPT);  // C is a multiple of CPT
  const TI* wp = w2t + cc;
  float w[DT_AHEAD][CPT];
#pragma unroll
  for (int k = 0; k < DT_AHEAD; ++k)
    if (warp + 8 * k < rank) get_cols<TI, CPT>(wp + (size_t)(warp + 8 * k) * C, w[k]);
  pdl_wait();
  const int t0 = blockIdx.y * TT, n = min(TT, T - t0);
  stage_tanh<TI, TT>(th, z + (long long)t0 * ld, ld, rank, n);
  __syncthreads();
  float acc[CPT][TT];
#pragma unroll
  for (int q = 0; q < CPT; ++q)
#pragma unroll
    for (int i = 0; i < TT; ++i) acc[q][i] = 0.f;
  auto add = [&](int j, const float (&wj)[CPT]) {
    float v[TT];
    get_tokens<TT>(th + j * TT, v);
#pragma unroll
    for (int q = 0; q < CPT; ++q)
#pragma unroll
      for (int i = 0; i < TT; ++i) acc[q][i] = fmaf(wj[q], v[i], acc[q][i]);
  };
#pragma unroll
  for (int k = 0; k < DT_AHEAD; ++k)
    if (warp + 8 * k < rank) add(warp + 8 * k, w[k]);
  for (int j = warp + 8 * DT_AHEAD; j < rank; j += 8) {
    get_cols<TI, CPT>(wp + (size_t)j * C, w[0]);
    add(j, w[0]);
  }
#pragma unroll
  for (int q = 0; q < CPT; ++q)
#pragma unroll
    for (int i = 0; i < TT; ++i) sums[(warp * TT + i) * COLS + lane + 32 * q] = acc[q][i];
  __syncthreads();
  for (int x = threadIdx.x; x < TT * COLS; x += 256) {
    const int i = x / COLS, s = x % COLS, col = (blockIdx.x * 32 + (s & 31)) * CPT + (s >> 5);
    float v = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) v += sums[(k * TT + i) * COLS + s];
    if (i < n && col < C) out[(long long)(t0 + i) * C + col] = expf(-expf(v + bias[col]));
  }
}

template <typename TO>
int launch_shift(const ShiftArgs& a, int T, bool vec, cudaStream_t s) {
  const int pieces = a.W / (vec ? 4 : 1);
  const int threads = pieces >= 512 && vec ? 512 : pieces >= 256 ? 256 : pieces >= 128 ? 128 : 64;
  const int nv = (pieces + threads - 1) / threads;
  // long portions: as many tokens a CTA as fill the SMs once (two CTAs an SM where a thread has one piece of a row); they
  // share the norms of their rows and what is read once a CTA
  const int slots = 148 * (nv == 1 ? 2 : 1), per = vec && T >= 1024 ? (T + slots - 1) / slots : 1;
  const dim3 grid((T + per - 1) / per), block(threads);
#define GO(V, NV, M, S) return launch_ex(shift_mix_kernel<TO, V, NV, M, S>, grid, block, 0, s, 1, a, T, per)
  if (!vec) GO(1, 0, 0, true);
  if (!a.token_seq) {
    if (nv == 1) GO(4, 1, 0, false);
    if (nv == 2) GO(4, 2, 0, false);
    if (nv <= 4) GO(4, 4, 0, false);
    GO(4, 0, 0, false);
  }
  if (nv == 1 && a.nmix == 5) GO(4, 1, 5, true);
  if (nv == 2 && a.nmix == 5) GO(4, 2, 5, true);
  if (nv <= 2) GO(4, 2, 0, true);
  if (nv <= 4) GO(4, 4, 0, true);
  GO(4, 0, 0, true);
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

// z: [T, >= rank] of type dt with row stride ld; w2t [rank, C] of type dt; bias float [C]; out float [T, C].
RLLM_API int rllm_lowrank_decay(int dt, const void* z, long long ld, int rank, const void* w2t, const float* bias, float* out,
                                int T, int C, void* stream) {
  if (T <= 0 || C <= 0) return 0;
  if (rank <= 0 || rank > DT_MAX_RANK) return ERR_BAD_SIZE;
  if (dt != DT_F32 && dt != DT_BF16) return ERR_BAD_DTYPE;
  if ((T + DT_TOKENS - 1) / DT_TOKENS > 65535) return ERR_TOO_LARGE;
  cudaStream_t s = (cudaStream_t)stream;
  const bool four = C % 4 == 0 && !((uintptr_t)w2t & 15) && !((uintptr_t)out & 15);
  if (T <= 16 * DT_TOKENS) {
    const int cpt = C % 2 == 0 ? 2 : 1;
    const dim3 grid((C + 32 * cpt - 1) / (32 * cpt), (T + DT_TOKENS - 1) / DT_TOKENS);
    const size_t smem = ((size_t)rank * DT_TOKENS + 8 * DT_TOKENS * 32 * cpt) * sizeof(float);      // at most 48 KB
#define GO(TI, N) return launch_ex(lowrank_decay_few_kernel<TI, N>, grid, dim3(256), smem, s, 1, (const TI*)z, ld, rank, (const TI*)w2t, bias, out, T, C)
    if (dt == DT_F32) { if (cpt == 2) GO(float, 2); GO(float, 1); }
    if (cpt == 2) GO(bf16, 2);
    GO(bf16, 1);
#undef GO
  }
  // tokens a tile: 16 where their shared memory and registers leave room
  const int cpt = four ? 4 : 1, tt = four && rank <= 512 ? 16 : 8;
  const dim3 grid((C + 128 * cpt - 1) / (128 * cpt), (T + tt - 1) / tt);
  const size_t smem = (size_t)rank * tt * sizeof(float);                                             // at most 32 KB
#define GO(TI, N, TT) return launch_ex(lowrank_decay_kernel<TI, N, TT>, grid, dim3(128), smem, s, 1, (const TI*)z, ld, rank, (const TI*)w2t, bias, out, T, C)
  if (dt == DT_F32) { if (tt == 16) GO(float, 4, 16); if (four) GO(float, 4, 8); GO(float, 1, 8); }
  if (tt == 16) GO(bf16, 4, 16);
  if (four) GO(bf16, 4, 8);
  GO(bf16, 1, 8);
#undef GO
}
