// What stands in front of a recurrence with token shift, float arithmetic throughout.
//
// shift_mix (one CTA a token): n = h / sqrt(mean(h^2) + eps) * w of the token's row and of the row before it in its
//   sequence (a portion's first token: the slot's `prev`, the normed row that the portion before ended with; no slot:
//   zeros), then `nmix` mixes n + (n_before - n) * mu_m, and optionally the plain row n and the same row under a
//   second norm's weight. The CTA of a portion's first token is the only one that touches its slot: having read
//   `prev` it writes the portion's last row there, which it norms itself, so that no CTA depends on another's order.
//   A row's norm is the same bits whichever CTA makes it. Without sequences (`token_seq` null) it is two norms of the
//   same rows in one pass.
// lowrank_decay: a = exp(-exp(W2 tanh(z) + b)) per column, z a row of `rank` numbers (the first projection's output). A thread
//   owns a column and walks the rank for eight tokens at a time, whose tanh(z) lie in shared memory.
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

template <typename TO, int VEC>
__global__ void shift_mix_kernel(const ShiftArgs a) {
  pdl_launch();
  pdl_wait();
  __shared__ float red[32];
  const int t = blockIdx.x, W = a.W, step = blockDim.x * VEC;
  const float* hr = a.h + (size_t)t * W;
  const float* other = nullptr;                      // the row before, or (a portion's first token) the portion's last row
  float* slot = nullptr;
  bool before = false;
  if (a.token_seq) {
    const int s = a.token_seq[t], row0 = a.cu_q[s], last = a.cu_q[s + 1] - 1;
    before = t > row0;
    const int id = !before && a.state_slots ? a.state_slots[s] : -1;
    if (id >= 0) slot = a.prev + (size_t)id * W;
    if (before) other = hr - W;
    else if (slot && last > t) other = a.h + (size_t)last * W;
  }
  auto root = [&](const float* row, float eps) {
    float ss = 0.f;
    for (int i = threadIdx.x * VEC; i < W; i += step) {
      float v[VEC];
      get<VEC>(row + i, v);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss = fmaf(v[e], v[e], ss);
    }
    ss = block_sum(ss, red) / (float)W;
    return make_float2(1.f / sqrtf(ss + eps), ss);
  };
  const float2 mine = root(hr, a.eps);
  const float r = mine.x, r2 = a.second ? 1.f / sqrtf(mine.y + a.eps2) : 0.f;
  const float ro = other ? root(other, a.eps).x : 0.f;
  for (int i = threadIdx.x * VEC; i < W; i += step) {
    float x[VEC], w[VEC], n[VEC], o[VEC], p[VEC], y[VEC];
    get<VEC>(hr + i, x);
    get<VEC>(a.w + i, w);
#pragma unroll
    for (int e = 0; e < VEC; ++e) { n[e] = x[e] * r * w[e]; o[e] = p[e] = 0.f; }
    if (other) {
      get<VEC>(other + i, o);
#pragma unroll
      for (int e = 0; e < VEC; ++e) o[e] = o[e] * ro * w[e];
    }
    if (before) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) p[e] = o[e];
    } else if (slot) {
      get<VEC>(slot + i, p);
      if (VEC == 1) slot[i] = other ? o[0] : n[0];
      else if (other) put<float, VEC>(slot + i, o);
      else put<float, VEC>(slot + i, n);
    }
    for (int m = 0; m < a.nmix; ++m) {
      float mu[VEC];
      get<VEC>(a.mu + (size_t)m * W + i, mu);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = fmaf(p[e] - n[e], mu[e], n[e]);
      put<TO, VEC>((TO*)a.mixes + ((size_t)t * a.nmix + m) * W + i, y);
    }
    if (a.plain) put<TO, VEC>((TO*)a.plain + (size_t)t * W + i, n);
    if (a.second) {
      get<VEC>(a.w2 + i, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = x[e] * r2 * w[e];
      put<TO, VEC>((TO*)a.second + (size_t)t * W + i, y);
    }
  }
}

constexpr int DT_TOKENS = 8, DT_MAX_RANK = 1024;

// VEC: W2's rows are read eight numbers at a time (rank a multiple of 8, rows on 16-byte boundaries).
template <typename TI, bool VEC>
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
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  float acc[DT_TOKENS];
#pragma unroll
  for (int i = 0; i < DT_TOKENS; ++i) acc[i] = 0.f;
  const TI* wr = w2 + (size_t)c * rank;
  auto walk = [&](float w, int j) {
    const float4 a = *reinterpret_cast<const float4*>(th + j * DT_TOKENS), b = *reinterpret_cast<const float4*>(th + j * DT_TOKENS + 4);
    acc[0] = fmaf(w, a.x, acc[0]); acc[1] = fmaf(w, a.y, acc[1]); acc[2] = fmaf(w, a.z, acc[2]); acc[3] = fmaf(w, a.w, acc[3]);
    acc[4] = fmaf(w, b.x, acc[4]); acc[5] = fmaf(w, b.y, acc[5]); acc[6] = fmaf(w, b.z, acc[6]); acc[7] = fmaf(w, b.w, acc[7]);
  };
  if (VEC) {
    for (int j = 0; j < rank; j += 8) {
      float w[8];
      if constexpr (sizeof(TI) == 2) {
        const uint4 u = *reinterpret_cast<const uint4*>(wr + j);
        const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
        for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(h2[e]); w[2 * e] = f.x; w[2 * e + 1] = f.y; }
      } else {
        const float4 u = *reinterpret_cast<const float4*>(wr + j), v = *reinterpret_cast<const float4*>(wr + j + 4);
        w[0] = u.x; w[1] = u.y; w[2] = u.z; w[3] = u.w; w[4] = v.x; w[5] = v.y; w[6] = v.z; w[7] = v.w;
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) walk(w[e], j + e);
    }
  } else {
    for (int j = 0; j < rank; ++j) walk(to_f32(wr[j]), j);
  }
  const float b = bias[c];
#pragma unroll
  for (int i = 0; i < DT_TOKENS; ++i)
    if (i < n) out[(long long)(t0 + i) * C + c] = expf(-expf(acc[i] + b));
}

template <typename TO>
int launch_shift(const ShiftArgs& a, int T, bool vec, cudaStream_t s) {
  const int per = a.W / (vec ? 4 : 1);
  const int threads = per >= 256 ? 256 : per >= 128 ? 128 : 64;
  return vec ? launch_ex(shift_mix_kernel<TO, 4>, dim3(T), dim3(threads), 0, s, 1, a)
             : launch_ex(shift_mix_kernel<TO, 1>, dim3(T), dim3(threads), 0, s, 1, a);
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
  const int threads = row_tiles >= 16 ? 128 : 32;     // few tokens: columns over more SMs
  const dim3 grid((C + threads - 1) / threads, row_tiles);
  const size_t smem = (size_t)rank * DT_TOKENS * sizeof(float);
  const bool vec = rank % 8 == 0 && !((uintptr_t)w2 & 15);
  cudaStream_t s = (cudaStream_t)stream;
#define GO(TI, V) return launch_ex(lowrank_decay_kernel<TI, V>, grid, dim3(threads), smem, s, 1, (const TI*)z, ld, rank, (const TI*)w2, bias, out, T, C)
  if (dt == DT_F32) { if (vec) GO(float, true); GO(float, false); }
  if (dt == DT_BF16) { if (vec) GO(bf16, true); GO(bf16, false); }
#undef GO
  return ERR_BAD_DTYPE;
}
