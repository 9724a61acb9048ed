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

template <typename T, int TOK>  // TOK tokens per block, TOK / LRD_TG per thread
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

// The same for bfloat16 prompts on the tensor cores (mma.sync m16n8k16): w2 is an exact operand, tanh(a) enters as two
// bfloat16 terms, rounded value and rounded rest, so the sums keep 16 bits of it or more.  A block: 64 tokens x 64 channels, a
// warp 16 of the tokens.
__device__ __forceinline__ void lrm_mma(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__global__ void __launch_bounds__(128)
low_rank_decay_mma_kernel(const __nv_bfloat16* __restrict__ a, long long a_stride, int tokens, int rank,
                          const __nv_bfloat16* __restrict__ w2, const float* __restrict__ w0, float* __restrict__ out,
                          int out_stride, int channels, int log_out) {
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, cp = (lane & 3) * 2;
  const int t0 = blockIdx.y * 64 + warp * 16, c0 = blockIdx.x * 64;
  float acc[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
  for (int k0 = 0; k0 < rank; k0 += 16) {
    unsigned ah[4], al[4];
#pragma unroll
    for (int q = 0; q < 4; ++q) {  // rows + 8 (q & 1), columns + 8 (q >> 1)
      const int t = t0 + g + 8 * (q & 1), k = k0 + cp + 8 * (q >> 1);
      float2 v = make_float2(0.f, 0.f);
      if (t < tokens && k < rank) {
        const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(a + (long long)t * a_stride + k);
        v = make_float2(tanhf(__bfloat162float(x.x)), tanhf(__bfloat162float(x.y)));
      }
      const __nv_bfloat162 h = __floats2bfloat162_rn(v.x, v.y);
      const __nv_bfloat162 l = __floats2bfloat162_rn(v.x - __bfloat162float(h.x), v.y - __bfloat162float(h.y));
      ah[q] = *reinterpret_cast<const unsigned*>(&h);
      al[q] = *reinterpret_cast<const unsigned*>(&l);
    }
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const int c = c0 + n * 8 + g;
      const __nv_bfloat16* wp = w2 + (long long)c * rank + k0 + cp;
      const unsigned b0 = c < channels && k0 + cp < rank ? *reinterpret_cast<const unsigned*>(wp) : 0u;
      const unsigned b1 = c < channels && k0 + cp + 8 < rank ? *reinterpret_cast<const unsigned*>(wp + 8) : 0u;
      lrm_mma(acc[n], ah, b0, b1);
      lrm_mma(acc[n], al, b0, b1);
    }
  }
#pragma unroll
  for (int n = 0; n < 8; ++n) {
    const int c = c0 + n * 8 + cp;
    if (c >= channels) continue;  // (channels are even here)
    const float2 b = *reinterpret_cast<const float2*>(w0 + c);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = t0 + g + 8 * h;
      if (t >= tokens) continue;
      float x = -expf(acc[n][2 * h] + b.x), y = -expf(acc[n][2 * h + 1] + b.y);
      if (!log_out) {
        x = expf(x);
        y = expf(y);
      }
      *reinterpret_cast<float2*>(out + (long long)t * out_stride + c) = make_float2(x, y);
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
  if (dtype == ULLM_DTYPE_BF16 && tokens > 16 && rank % 2 == 0 && a_stride % 2 == 0 && channels % 2 == 0 && out_stride % 2 == 0 &&
      (((uintptr_t)a | (uintptr_t)w2) & 3) == 0 && (((uintptr_t)w0 | (uintptr_t)out) & 7) == 0 && (tokens + 63) / 64 <= 65535)
    return ullm_launch_kernel(low_rank_decay_mma_kernel, dim3((channels + 63) / 64, (tokens + 63) / 64), dim3(128), 0, st,
                              (const __nv_bfloat16*)a, a_stride, tokens, rank, (const __nv_bfloat16*)w2, w0, out, out_stride,
                              channels, log_out);
  const int tok = tokens <= 16 ? 4 : 32;
  const dim3 grid((channels + LRD_C - 1) / LRD_C, (tokens + tok - 1) / tok), block(LRD_C * LRD_TG);
  if (grid.y > 65535) return ULLM_ERR_UNSUPPORTED;
#define LR_GO(T)                                                                                                       \
  {                                                                                                                    \
    if (tok == 4)                                                                                                      \
      return ullm_launch_kernel(low_rank_decay_kernel<T, 4>, grid, block, 0, st, (const T*)a, a_stride, tokens, rank,   \
                                (const T*)w2, w0, out, out_stride, channels, log_out);                                 \
    return ullm_launch_kernel(low_rank_decay_kernel<T, 32>, grid, block, 0, st, (const T*)a, a_stride, tokens, rank,    \
                              (const T*)w2, w0, out, out_stride, channels, log_out);                                   \
  }
  if (dtype == ULLM_DTYPE_F32) LR_GO(float);
  if (dtype == ULLM_DTYPE_BF16) LR_GO(__nv_bfloat16);
  if (dtype == ULLM_DTYPE_F16) LR_GO(__half);
#undef LR_GO
  return ULLM_ERR_BAD_DTYPE;
}
