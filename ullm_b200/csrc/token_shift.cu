// What stands in front of a recurrence that reads mixes of every row with the row before it, and takes its decays from a
// low-rank projection:
//
//   token_shift_mix   out[g][t] = h[t] + (h[t - 1] - h[t]) * mu[g]     for G mixes of the same rows at once
//   low_rank_decay    out[t][c] = exp(-exp(w2[c] . tanh(a[t]) + w0[c]))   (or its logarithm), all in 32-bit
//
// The row in front of a request's first token of the step comes from its state row (32-bit; zeros for a new request).  In a
// step of single tokens the thread that reads a channel of it is its only reader and moves it on; otherwise
// `conv_state_update` (csrc/attention_prep.cu, two taps) does so behind this kernel.
#include "common.cuh"

#define TSH_MAX_MIXES 16

template <typename T, int VEC>
__global__ void token_shift_mix_kernel(const T* __restrict__ h, long long h_stride, const float* __restrict__ mu, int mixes,
                                       int width, T* __restrict__ out, float* __restrict__ state, long long state_stride,
                                       int num_slots, const int* __restrict__ cu_q, const int* __restrict__ token_req,
                                       const int* __restrict__ req_slots, int tokens, int single, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.y;
  const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (c0 >= width) return;
  float x[VEC], d[VEC], m[VEC];
  load_vec<T, VEC>(h + (long long)t * h_stride + c0, x);
#pragma unroll
  for (int i = 0; i < VEC; ++i) d[i] = 0.f;
  const int r = token_req[t];
  if (r >= 0) {
    if (t > cu_q[r]) {
      load_vec<T, VEC>(h + (long long)(t - 1) * h_stride + c0, d);
    } else {
      const int slot = req_slots[r];
      if (slot >= 0 && slot < num_slots) {
        float* st = state + (long long)slot * state_stride + c0;
        load_vec32<VEC>(st, d);
        if (single) store_vec32<VEC>(st, x);
      } else if (c0 == 0) {
        ullm_report(status, ULLM_STATUS_SLOT, t, slot);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < VEC; ++i) d[i] -= x[i];
  for (int g = 0; g < mixes; ++g) {
    load_vec32<VEC>(mu + (long long)g * width + c0, m);
#pragma unroll
    for (int i = 0; i < VEC; ++i) m[i] = fmaf(d[i], m[i], x[i]);
    store_vec<T, VEC>(out + ((long long)g * tokens + t) * width + c0, m);
  }
}

// A block: LRD_C channels x LRD_T tokens, LRD_R of the rank at a time; a thread: one channel and LRD_T / LRD_TG tokens.
#define LRD_C 64
#define LRD_TG 4
#define LRD_R 32

template <typename T, int TOK>  // TOK tokens per block, TOK / LRD_TG per thread (steps of few tokens)
__global__ void __launch_bounds__(LRD_C * LRD_TG)
low_rank_decay_kernel(const T* __restrict__ a, long long a_stride, int tokens, int rank, const T* __restrict__ w2,
                      const float* __restrict__ w0, float* __restrict__ out, int out_stride, int channels, int log_out) {
  constexpr int PER = TOK / LRD_TG;
  __shared__ float w_s[LRD_C][LRD_R + 1];
  __shared__ float a_s[TOK][LRD_R];
  pdl_launch_dependents();
  pdl_wait();
  const int c0 = blockIdx.x * LRD_C, t0 = blockIdx.y * TOK;
  const int c = threadIdx.x % LRD_C, tg = threadIdx.x / LRD_C;
  float acc[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) acc[i] = 0.f;
  for (int r0 = 0; r0 < rank; r0 += LRD_R) {
    const int n = min(LRD_R, rank - r0);
    for (int i = threadIdx.x; i < LRD_C * LRD_R; i += LRD_C * LRD_TG) {
      const int cc = i / LRD_R, r = i - cc * LRD_R;
      w_s[cc][r] = (c0 + cc < channels && r < n) ? to_f32(w2[(long long)(c0 + cc) * rank + r0 + r]) : 0.f;
    }
    for (int i = threadIdx.x; i < TOK * LRD_R; i += LRD_C * LRD_TG) {
      const int tt = i / LRD_R, r = i - tt * LRD_R;
      a_s[tt][r] = (t0 + tt < tokens && r < n) ? tanhf(to_f32(a[(long long)(t0 + tt) * a_stride + r0 + r])) : 0.f;
    }
    __syncthreads();
#pragma unroll 4
    for (int r = 0; r < LRD_R; ++r) {
      const float w = w_s[c][r];
#pragma unroll
      for (int i = 0; i < PER; ++i) acc[i] = fmaf(w, a_s[tg * PER + i][r], acc[i]);
    }
    __syncthreads();
  }
  if (c0 + c >= channels) return;
  const float b = w0[c0 + c];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int t = t0 + tg * PER + i;
    if (t >= tokens) return;
    const float l = -expf(acc[i] + b);
    out[(long long)t * out_stride + c0 + c] = log_out ? l : expf(l);
  }
}

// The same for prompts: a block of 128 channels x 64 tokens, a thread eight by four, so that three 16-byte reads of shared
// memory serve 32 multiply-adds and every tanh is formed once per 128 channels.
#define LRP_TILE 64
#define LRP_C 128
template <typename T>
__global__ void __launch_bounds__(256)
low_rank_decay_tiled_kernel(const T* __restrict__ a, long long a_stride, int tokens, int rank, const T* __restrict__ w2,
                            const float* __restrict__ w0, float* __restrict__ out, int out_stride, int channels, int log_out) {
  __shared__ __align__(16) float w_s[LRD_R][LRP_C + 4];
  __shared__ __align__(16) float a_s[LRD_R][LRP_TILE + 4];
  pdl_launch_dependents();
  pdl_wait();
  const int c0 = blockIdx.x * LRP_C, t0 = blockIdx.y * LRP_TILE;
  const int c = (threadIdx.x & 15) * 4, t = (threadIdx.x >> 4) * 4;  // channels c .. c + 3 and c + 64 .. c + 67
  float acc[4][8];  // [token][channel]
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[i][j] = 0.f;
  for (int r0 = 0; r0 < rank; r0 += LRD_R) {
    const int n = min(LRD_R, rank - r0);
    for (int i = threadIdx.x; i < LRP_C * LRD_R; i += 256) {
      const int row = i / LRD_R, r = i - row * LRD_R;
      w_s[r][row] = (c0 + row < channels && r < n) ? to_f32(w2[(long long)(c0 + row) * rank + r0 + r]) : 0.f;
    }
    for (int i = threadIdx.x; i < LRP_TILE * LRD_R; i += 256) {
      const int row = i / LRD_R, r = i - row * LRD_R;
      a_s[r][row] = (t0 + row < tokens && r < n) ? tanhf(to_f32(a[(long long)(t0 + row) * a_stride + r0 + r])) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int r = 0; r < LRD_R; ++r) {
      const float4 w = *reinterpret_cast<const float4*>(&w_s[r][c]), w4 = *reinterpret_cast<const float4*>(&w_s[r][c + 64]),
                   x = *reinterpret_cast<const float4*>(&a_s[r][t]);
      const float wv[8] = {w.x, w.y, w.z, w.w, w4.x, w4.y, w4.z, w4.w}, xv[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[i][j] = fmaf(wv[j], xv[i], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int ch = c0 + c + 64 * h;
    if (ch >= channels) return;
    float b[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) b[j] = ch + j < channels ? w0[ch + j] : 0.f;
    const bool wide = (out_stride & 3) == 0 && ch + 4 <= channels && (reinterpret_cast<uintptr_t>(out) & 15) == 0;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      if (t0 + t + i >= tokens) break;
      float v[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float l = -expf(acc[i][4 * h + j] + b[j]);
        v[j] = log_out ? l : expf(l);
      }
      float* dst = out + (long long)(t0 + t + i) * out_stride + ch;
      if (wide) {
        *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (ch + j < channels) dst[j] = v[j];
      }
    }
  }
}

template <typename T>
static int shift_go(const void* h, long long h_stride, const float* mu, int mixes, int width, void* out, float* state,
                    long long state_stride, int num_slots, const int* cu_q, const int* token_req, const int* req_slots,
                    int tokens, int single, int* status, cudaStream_t st) {
  constexpr int V = 16 / (int)sizeof(T);
  const bool wide = width % V == 0 && h_stride % V == 0 && state_stride % 4 == 0 &&
                    (((uintptr_t)h | (uintptr_t)mu | (uintptr_t)out | (uintptr_t)state) & 15) == 0;
  const int vec = wide ? V : 1;
  int threads = 32;
  while (threads < 256 && threads * vec < width) threads <<= 1;
  const dim3 grid((width + threads * vec - 1) / (threads * vec), tokens), block(threads);
  if (wide)
    return ullm_launch_kernel(token_shift_mix_kernel<T, V>, grid, block, 0, st, (const T*)h, h_stride, mu, mixes, width,
                              (T*)out, state, state_stride, num_slots, cu_q, token_req, req_slots, tokens, single, status);
  return ullm_launch_kernel(token_shift_mix_kernel<T, 1>, grid, block, 0, st, (const T*)h, h_stride, mu, mixes, width, (T*)out,
                            state, state_stride, num_slots, cu_q, token_req, req_slots, tokens, single, status);
}

// h [tokens, width] (rows `h_stride` apart), mu [mixes][width] 32-bit, out [mixes][tokens][width]; state: 32-bit rows of
// `width` floats, `state_stride` apart.  `single`: every request of the step has one token.
extern "C" int ullm_token_shift_mix(int dtype, const void* h, long long h_stride, const float* mu, int mixes, int width,
                                    void* out, float* state, long long state_stride, int num_slots, const int* cu_q,
                                    const int* token_req, const int* req_slots, int tokens, int single, int* status,
                                    void* stream) {
  cudaStream_t st = (cudaStream_t)stream;
  if (tokens < 0 || width <= 0 || mixes <= 0 || h_stride < width || state_stride < width || num_slots <= 0)
    return ULLM_ERR_BAD_SIZE;
  if (mixes > TSH_MAX_MIXES || tokens > 65535) return ULLM_ERR_UNSUPPORTED;
  if (tokens == 0) return ULLM_OK;
#define TS_ARGS h, h_stride, mu, mixes, width, out, state, state_stride, num_slots, cu_q, token_req, req_slots, tokens, single, status, st
  if (dtype == ULLM_DTYPE_F32) return shift_go<float>(TS_ARGS);
  if (dtype == ULLM_DTYPE_BF16) return shift_go<__nv_bfloat16>(TS_ARGS);
  if (dtype == ULLM_DTYPE_F16) return shift_go<__half>(TS_ARGS);
#undef TS_ARGS
  return ULLM_ERR_BAD_DTYPE;
}

// a [tokens, rank] (rows `a_stride` apart), w2 [channels, rank], w0 [channels] 32-bit, out [tokens, channels] 32-bit (rows
// `out_stride` apart).
extern "C" int ullm_low_rank_decay(int dtype, const void* a, long long a_stride, int tokens, int rank, const void* w2,
                                   const float* w0, float* out, int out_stride, int channels, int log_out, void* stream) {
  cudaStream_t st = (cudaStream_t)stream;
  if (tokens < 0 || rank <= 0 || channels <= 0 || a_stride < rank || out_stride < channels) return ULLM_ERR_BAD_SIZE;
  if (tokens == 0) return ULLM_OK;
  const int tok = tokens <= 16 ? 4 : LRP_TILE;
  const int cb = tok == 4 ? LRD_C : LRP_C;
  const dim3 grid((channels + cb - 1) / cb, (tokens + tok - 1) / tok), block(LRD_C * LRD_TG);
  if (grid.y > 65535) return ULLM_ERR_UNSUPPORTED;
#define LR_GO(T)                                                                                                       \
  {                                                                                                                    \
    if (tok == 4)                                                                                                      \
      return ullm_launch_kernel(low_rank_decay_kernel<T, 4>, grid, block, 0, st, (const T*)a, a_stride, tokens, rank,   \
                                (const T*)w2, w0, out, out_stride, channels, log_out);                                 \
    return ullm_launch_kernel(low_rank_decay_tiled_kernel<T>, grid, block, 0, st, (const T*)a, a_stride, tokens, rank,  \
                              (const T*)w2, w0, out, out_stride, channels, log_out);                                   \
  }
  if (dtype == ULLM_DTYPE_F32) LR_GO(float);
  if (dtype == ULLM_DTYPE_BF16) LR_GO(__nv_bfloat16);
  if (dtype == ULLM_DTYPE_F16) LR_GO(__half);
#undef LR_GO
  return ULLM_ERR_BAD_DTYPE;
}
