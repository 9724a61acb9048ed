// A state-space recurrence with a scalar decay per head ("state-space duality", Mamba-2), for any mix of requests in one
// flat batch: prompt portions of any length beside single decoded tokens.
//
//   ssd_prepare     from the projection's rows [.. | x B C | dt]: the causal convolution over time of every channel of
//                   x | B | C with a bias, then silu (rounded to the engine's dtype), and per head, in 32-bit,
//                   dt = softplus(dt_raw + dt_bias) and the logarithm of the decay, -exp(A_log) dt
//   ssd_recurrence  per request and head, S [N, P] in 32-bit, kept in the request's state row between steps:
//                     S_t = exp(-exp(A_log) dt_t) S_{t-1} + dt_t B_t x_t^T,    y_t = S_t^T C_t + D x_t
//                   (head h reads B and C of group h / (heads / groups))
//   ssd_gate_norm   y <- y * silu(z), then every one of `parts` equal stretches of the row divided by its own root mean
//                   square, times a weight per channel; or the norm first and sigmoid(z) behind it
//
// Steps and decays that do not depend on the token (a linear attention with a fixed decay per head: x = v, B = k, C = q,
// dt = 1) come as one row with a row stride of 0; `silu_in` puts a silu on x, B and C as they are read.
//
// The taps - 1 projected rows in front of a step's first token come from the state row too (zeros for a new request);
// in a decode step `ssd_prepare` moves them on itself, otherwise `conv_state_update` (csrc/attention_prep.cu) after it.  The recurrence runs token by token in a
// fixed order, so a request's result does not depend on how its tokens were cut into steps or on what else is in the
// batch.  Its parallelism is over requests, heads and the columns of S: a block owns (request, head, a tile of
// columns); a column's N rows are spread over `rs` neighbouring lanes in pieces of four, which meet in shuffles for
// the read-out.  B, C, x and the decays of a chunk of tokens are staged in shared memory by a second set of threads
// while the first set runs the chunk before (two buffers).
//
// State row layout (floats): S^T as [heads][P][N], then the convolution's rows [taps - 1][channels].
#include "common.cuh"

#define SSD_THREADS 128  // threads that run the recurrence; as many again stage the next chunk
#define SSD_MAX_STATE 512
#define SSD_MAX_TAPS 32

__device__ __forceinline__ float ssd_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

// One thread: VEC neighbouring channels of TOK tokens in a row.  With TAPS > 0 (the usual counts as constants) the filter
// and the taps - 1 rows in front of the current token wait in registers, so every row is read once.  The blocks behind the
// channels' (blockIdx.x >= channel_blocks) do the step sizes.  `single`: every request of the step has one token; the
// thread that convolves a channel is then the only reader of its memory and moves it on itself.
template <typename T, int VEC, int TAPS, int TOK>
__global__ void ssd_prepare_kernel(const T* __restrict__ u, long long row_stride, int xbc_off, int dt_off, int channels,
                                   int heads, const T* __restrict__ conv_w, int taps_rt,
                                   const float* __restrict__ conv_b, const float* __restrict__ dt_bias,
                                   const float* __restrict__ a_log, float* __restrict__ conv_state,
                                   long long state_stride, int num_slots, const int* __restrict__ cu_q,
                                   const int* __restrict__ token_req, const int* __restrict__ req_slots, int tokens,
                                   T* __restrict__ xbc, float* __restrict__ dt, float* __restrict__ log_decay,
                                   int channel_blocks, int single, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int taps = TAPS > 0 ? TAPS : taps_rt;
  const int tok0 = blockIdx.y * TOK, tok1 = min(tokens, tok0 + TOK);
  if ((int)blockIdx.x >= channel_blocks) {
    const int h = (blockIdx.x - channel_blocks) * blockDim.x + threadIdx.x;
    if (h >= heads) return;
    const float neg_a = -expf(a_log[h]), bias = dt_bias[h];
    for (int t = tok0; t < tok1; ++t) {
      const float d = token_req[t] >= 0 ? ssd_softplus(to_f32(u[(long long)t * row_stride + dt_off + h]) + bias) : 0.f;
      dt[(long long)t * heads + h] = d;
      log_decay[(long long)t * heads + h] = neg_a * d;
    }
    return;
  }
  const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (c0 >= channels) return;
  float cur[TOK][VEC];  // (asked for before anything depends on them)
#pragma unroll
  for (int i = 0; i < TOK; ++i)
    if (tok0 + i < tok1) load_vec<T, VEC>(u + (long long)(tok0 + i) * row_stride + xbc_off + c0, cur[i]);
  constexpr int TW = TAPS > 0 ? TAPS : 1, BACK = TAPS > 1 ? TAPS - 1 : 1;
  float w[TW][VEC];  // flat: element i * TAPS + j is channel c0 + i's tap j
  if (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TW; ++j) load_vec<T, VEC>(conv_w + (long long)c0 * TW + j * VEC, w[j]);
  }
  float bias[VEC], win[BACK][VEC];
  load_vec32<VEC>(conv_b + c0, bias);
  int prev = -1, t0 = 0;
  float* st = nullptr;
#pragma unroll
  for (int i = 0; i < TOK; ++i) {
    const int t = tok0 + i;
    if (t >= tok1) break;
    const int r = token_req[t];
    float y[VEC];
    if (r < 0) {  // a row that belongs to no request
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = 0.f;
      store_vec<T, VEC>(xbc + (long long)t * channels + c0, y);
      prev = -1;
      continue;
    }
    const bool fresh = r != prev;
    if (fresh) {
      prev = r;
      t0 = cu_q[r];
      const int slot = req_slots[r];
      st = nullptr;
      if (taps > 1 && slot >= 0 && slot < num_slots) st = conv_state + (long long)slot * state_stride + c0;
      else if (taps > 1) ullm_report(status, ULLM_STATUS_SLOT, t, slot);
    }
    auto row_back = [&](int back, float(&v)[VEC]) {  // the projected row `back` >= 1 tokens before t
      if (t - back >= t0) {
        load_vec<T, VEC>(u + (long long)(t - back) * row_stride + xbc_off + c0, v);
      } else if (st != nullptr) {
        load_vec32<VEC>(st + (long long)(taps - 1 - (t0 - (t - back))) * channels, v);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = 0.f;
      }
    };
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = bias[e];
    if (TAPS > 0) {
      if (fresh && TAPS > 1) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) row_back(TAPS - 1 - j, win[j]);
      }
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          const int f = e * TW + j;  // (f / VEC, f % VEC: constants after unrolling)
          y[e] = fmaf(w[f / VEC][f % VEC], j < TAPS - 1 ? win[j < BACK ? j : 0][e] : cur[i][e], y[e]);
        }
      }
      if (TAPS > 1) {
#pragma unroll
        for (int j = 0; j + 1 < TAPS - 1; ++j)
#pragma unroll
          for (int e = 0; e < VEC; ++e) win[j][e] = win[j + 1][e];
#pragma unroll
        for (int e = 0; e < VEC; ++e) win[BACK - 1][e] = cur[i][e];
        if (single && st != nullptr) {
#pragma unroll
          for (int j = 0; j < TAPS - 1; ++j) store_vec32<VEC>(st + (long long)j * channels, win[j]);
        }
      }
    } else {
      float v[VEC];
      for (int j = 0; j < taps - 1; ++j) {
        row_back(taps - 1 - j, v);
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = fmaf(to_f32(conv_w[(long long)(c0 + e) * taps + j]), v[e], y[e]);
        if (single && st != nullptr && j > 0) store_vec32<VEC>(st + (long long)(j - 1) * channels, v);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = fmaf(to_f32(conv_w[(long long)(c0 + e) * taps + taps - 1]), cur[i][e], y[e]);
      if (single && st != nullptr) store_vec32<VEC>(st + (long long)(taps - 2) * channels, cur[i]);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = act_silu(y[e]);
    store_vec<T, VEC>(xbc + (long long)t * channels + c0, y);
  }
}

// Threads 0 .. 127 run the recurrence on the chunk of tokens in one half of shared memory while threads 128 .. 255 stage
// the next chunk in the other half.  A staged row of B and C is padded with zeros to RPT * rs entries, so the row loop
// has no bounds checks: the padded rows of S stay zero.  CPT: neighbouring columns a thread holds.
template <typename T, int RPT, int CPT>
__global__ void __launch_bounds__(2 * SSD_THREADS)
ssd_recurrence_kernel(const T* __restrict__ xbc, long long row_stride, int b_off, int c_off,
                      const float* __restrict__ dt, const float* __restrict__ log_decay, const float* __restrict__ d_skip,
                      float* __restrict__ state, long long state_stride, const int* __restrict__ cu_q,
                      const int* __restrict__ req_slots, const int* __restrict__ token_req, float* __restrict__ out,
                      int heads, int n_state, int pdim, int per_group, int rs, int chunk, int num_slots, int most_tokens,
                      int* status, long long dt_stride, int silu_in) {
  extern __shared__ __align__(16) float sm[];
  pdl_launch_dependents();
  pdl_wait();
  const int req = blockIdx.z, head = blockIdx.y;
  const int groups = SSD_THREADS / rs;  // column groups of a block
  const int cols_per_block = groups * CPT;
  const bool loader = threadIdx.x >= SSD_THREADS;
  const int tid = threadIdx.x & (SSD_THREADS - 1);
  const int lane_row = tid % rs, group = tid / rs;
  const int col0 = blockIdx.x * cols_per_block;
  const int col = col0 + group * CPT;
  const int dimp = RPT * rs;
  const int t0 = cu_q[req], t1 = cu_q[req + 1];
  if (t1 <= t0 || t1 - t0 > most_tokens) return;  // (longer portions are another kernel's)
  if (token_req[t0] < 0) {  // a row that belongs to no request: zeros out, no state touched
    if (!loader && lane_row == 0)
      for (int t = t0; t < t1; ++t)
        for (int c = 0; c < CPT; ++c)
          if (col + c < pdim) out[((long long)t * heads + head) * pdim + col + c] = 0.f;
    return;
  }
  const int slot = req_slots[req];
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0) ullm_report(status, ULLM_STATUS_SLOT, req, slot);
    return;
  }
  const int buf_floats = chunk * (2 * dimp + cols_per_block + 4);
  float* st_head = state + (long long)slot * state_stride + (long long)head * pdim * n_state;
  const int x_off = head * pdim;
  const int bg = b_off + (head / per_group) * n_state, cg = c_off + (head / per_group) * n_state;
  const bool vec8 = sizeof(T) == 2 && (n_state & 7) == 0 && (dimp & 7) == 0 && (bg & 7) == 0 && (cg & 7) == 0 &&
                    (row_stride & 7) == 0 && (reinterpret_cast<uintptr_t>(xbc) & 15) == 0;

  auto fill = [&](int which, int c0, int cn) {  // loader threads: tokens c0 .. c0 + cn - 1 into buffer `which`
    float* sb = sm + which * buf_floats;  // [chunk][dimp]
    float* sc = sb + chunk * dimp;
    float* sx = sc + chunk * dimp;        // [chunk][cols_per_block]: dt * x
    float* ss = sx + chunk * cols_per_block;  // [chunk][4]: decay
    if (vec8) {
      const int per_tok = dimp >> 3, n8 = cn * per_tok;
      for (int g = tid; g < n8; g += SSD_THREADS) {
        const int t = g / per_tok, r = (g - t * per_tok) << 3;
        float vb[8], vc[8];
        if (r < n_state) {
          load_vec<T, 8>(xbc + (long long)(c0 + t) * row_stride + bg + r, vb);
          load_vec<T, 8>(xbc + (long long)(c0 + t) * row_stride + cg + r, vc);
          if (silu_in) {
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              vb[i] = act_silu(vb[i]);
              vc[i] = act_silu(vc[i]);
            }
          }
        } else {
#pragma unroll
          for (int i = 0; i < 8; ++i) vb[i] = vc[i] = 0.f;
        }
        store_vec32<8>(sb + (g << 3), vb);
        store_vec32<8>(sc + (g << 3), vc);
      }
    } else {
      for (int i = tid; i < cn * dimp; i += SSD_THREADS) {
        const int t = i / dimp, r = i - t * dimp;
        const T* row = xbc + (long long)(c0 + t) * row_stride;
        float b = r < n_state ? to_f32(row[bg + r]) : 0.f, c = r < n_state ? to_f32(row[cg + r]) : 0.f;
        if (silu_in) {  // (silu(0) = 0: the padding stays zero)
          b = act_silu(b);
          c = act_silu(c);
        }
        sb[i] = b;
        sc[i] = c;
      }
    }
    for (int i = tid; i < cn * cols_per_block; i += SSD_THREADS) {
      const int t = i / cols_per_block, c = i - t * cols_per_block;
      const float x = col0 + c < pdim ? to_f32(xbc[(long long)(c0 + t) * row_stride + x_off + col0 + c]) : 0.f;
      sx[i] = silu_in ? act_silu(x) : x;
    }
    for (int t = tid; t < cn; t += SSD_THREADS) {
      ss[t * 4] = expf(log_decay[(long long)(c0 + t) * dt_stride + head]);
      ss[t * 4 + 1] = dt[(long long)(c0 + t) * dt_stride + head];
    }
  };

  const bool s4 = (n_state & 3) == 0 && (reinterpret_cast<uintptr_t>(st_head) & 15) == 0;
  float S[RPT][CPT];
  if (!loader) {
#pragma unroll
    for (int g = 0; g < RPT / 4; ++g) {
      const int r = (g * rs + lane_row) * 4;
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        const float* p = st_head + (long long)(col + c) * n_state + r;
        if (s4 && col + c < pdim && r < n_state) {
          const float4 v = *reinterpret_cast<const float4*>(p);
          S[4 * g][c] = v.x;
          S[4 * g + 1][c] = v.y;
          S[4 * g + 2][c] = v.z;
          S[4 * g + 3][c] = v.w;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) S[4 * g + e][c] = (col + c < pdim && r + e < n_state) ? p[e] : 0.f;
        }
      }
    }
  } else {
    fill(0, t0, min(chunk, t1 - t0));
  }
  const float skip = d_skip[head];
  __syncthreads();
  int which = 0;
  for (int c0 = t0; c0 < t1; c0 += chunk, which ^= 1) {
    const int cn = min(chunk, t1 - c0);
    if (loader) {
      if (c0 + chunk < t1) fill(which ^ 1, c0 + chunk, min(chunk, t1 - c0 - chunk));
    } else {
      const float* sb = sm + which * buf_floats;
      const float* sc = sb + chunk * dimp;
      const float* sx = sc + chunk * dimp;
      const float* ss = sx + chunk * cols_per_block;
      // four tokens share one chain of shuffles: only S carries a dependence from token to token
      constexpr int TB = 4;
      for (int t = 0; t < cn; t += TB) {
        float acc[TB][CPT];
#pragma unroll
        for (int j = 0; j < TB; ++j) {
#pragma unroll
          for (int c = 0; c < CPT; ++c) acc[j][c] = 0.f;
          if (t + j < cn) {
            const float a = ss[(t + j) * 4], d = ss[(t + j) * 4 + 1];
            float x[CPT];
#pragma unroll
            for (int c = 0; c < CPT; ++c) x[c] = d * sx[(t + j) * cols_per_block + group * CPT + c];
            const float4* b4 = reinterpret_cast<const float4*>(sb + (t + j) * dimp) + lane_row;
            const float4* c4 = reinterpret_cast<const float4*>(sc + (t + j) * dimp) + lane_row;
#pragma unroll
            for (int g = 0; g < RPT / 4; ++g) {
              const float4 bv = b4[g * rs], cv = c4[g * rs];
              const float br[4] = {bv.x, bv.y, bv.z, bv.w}, cr[4] = {cv.x, cv.y, cv.z, cv.w};
#pragma unroll
              for (int e = 0; e < 4; ++e) {
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                  S[4 * g + e][c] = fmaf(a, S[4 * g + e][c], br[e] * x[c]);
                  acc[j][c] = fmaf(S[4 * g + e][c], cr[e], acc[j][c]);
                }
              }
            }
          }
        }
        for (int o = rs >> 1; o > 0; o >>= 1) {
#pragma unroll
          for (int j = 0; j < TB; ++j)
#pragma unroll
            for (int c = 0; c < CPT; ++c) acc[j][c] += __shfl_xor_sync(0xffffffffu, acc[j][c], o);
        }
        if (lane_row == 0) {
#pragma unroll
          for (int j = 0; j < TB; ++j)
            if (t + j < cn) {
#pragma unroll
              for (int c = 0; c < CPT; ++c)
                if (col + c < pdim)
                  out[((long long)(c0 + t + j) * heads + head) * pdim + col + c] =
                      fmaf(skip, sx[(t + j) * cols_per_block + group * CPT + c], acc[j][c]);
            }
        }
      }
    }
    __syncthreads();  // the next chunk is staged, this one has been read
  }
  if (!loader) {
#pragma unroll
    for (int g = 0; g < RPT / 4; ++g) {
      const int r = (g * rs + lane_row) * 4;
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        float* p = st_head + (long long)(col + c) * n_state + r;
        if (s4 && col + c < pdim && r < n_state) {
          *reinterpret_cast<float4*>(p) = make_float4(S[4 * g][c], S[4 * g + 1][c], S[4 * g + 2][c], S[4 * g + 3][c]);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (col + c < pdim && r + e < n_state) p[e] = S[4 * g + e][c];
        }
      }
    }
  }
}

// One block per (token, part): g = y silu(z) waits in shared memory for the part's sum of squares.
template <typename T, int VEC>
__global__ void ssd_gate_norm_kernel(const float* __restrict__ y, const T* __restrict__ z, long long z_stride,
                                     const float* __restrict__ w, T* __restrict__ out, int inner, int part_size,
                                     float eps, int gate_behind) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float scratch[33];
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  const int p0 = blockIdx.y * part_size;
  float sq = 0.f;
  for (int c = threadIdx.x * VEC; c < part_size; c += blockDim.x * VEC) {
    float g[VEC], zv[VEC];
    load_vec32<VEC>(y + t * inner + p0 + c, g);
    load_vec<T, VEC>(z + t * z_stride + p0 + c, zv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      if (!gate_behind) g[i] *= act_silu(zv[i]);
      sq += g[i] * g[i];
    }
    store_vec32<VEC>(sm + c, g);
  }
  const float rstd = 1.f / sqrtf(block_sum(sq, scratch) / (float)part_size + eps);
  for (int c = threadIdx.x * VEC; c < part_size; c += blockDim.x * VEC) {  // (a thread reads what it wrote itself)
    float g[VEC], wv[VEC];
    load_vec32<VEC>(sm + c, g);
    load_vec32<VEC>(w + p0 + c, wv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) g[i] *= rstd * wv[i];
    if (gate_behind) {
      float zv[VEC];
      load_vec<T, VEC>(z + t * z_stride + p0 + c, zv);
#pragma unroll
      for (int i = 0; i < VEC; ++i) g[i] /= 1.f + expf(-zv[i]);
    }
    store_vec<T, VEC>(out + t * inner + p0 + c, g);
  }
}

extern "C" int ullm_ssd_supported(int heads, int n_state, int pdim, int groups, int taps) {
  return heads > 0 && n_state > 0 && pdim > 0 && groups > 0 && heads % groups == 0 && n_state <= SSD_MAX_STATE &&
         taps >= 1 && taps <= SSD_MAX_TAPS && heads <= 65535;
}

template <typename T>
static int prepare_go(const void* u, long long row_stride, int xbc_off, int dt_off, int channels, int heads,
                      const void* conv_w, int taps, const float* conv_b, const float* dt_bias, const float* a_log,
                      float* conv_state, long long state_stride, int num_slots, const int* cu_q,
                      const int* token_req, const int* req_slots, int tokens, void* xbc, float* dt, float* log_decay,
                      int single, int* status, cudaStream_t st) {
  constexpr int V = 16 / (int)sizeof(T);
  const bool wide = channels % V == 0 && xbc_off % V == 0 && row_stride % V == 0 && state_stride % 4 == 0 &&
                    (((uintptr_t)u | (uintptr_t)xbc | (uintptr_t)conv_state | (uintptr_t)conv_w | (uintptr_t)conv_b) & 15) == 0;
  const int vec = wide ? V : 1;
  // steps of few tokens: a token per thread; prompts: four tokens share a thread's filter and rows (2 and 8: 10 % slower)
  const int tok = tokens >= 512 ? 4 : 1, threads = 64;
  const int cb = (channels + threads * vec - 1) / (threads * vec), hb = (heads + threads - 1) / threads;
  const dim3 grid(cb + hb, (tokens + tok - 1) / tok), block(threads);
  if (grid.y > 65535) return ULLM_ERR_BAD_SIZE;
#define SP_GO(VEC, TAPS, TOK)                                                                                         \
  return ullm_launch_kernel(ssd_prepare_kernel<T, VEC, TAPS, TOK>, grid, block, 0, st, (const T*)u, row_stride,       \
                            xbc_off, dt_off, channels, heads, (const T*)conv_w, taps, conv_b, dt_bias, a_log,         \
                            conv_state, state_stride, num_slots, cu_q, token_req, req_slots, tokens, (T*)xbc, dt,     \
                            log_decay, cb, single, status)
#define SP_TOK(VEC, TAPS)              \
  {                                    \
    if (tok == 4) SP_GO(VEC, TAPS, 4); \
    SP_GO(VEC, TAPS, 1);               \
  }
  if (wide) {
    if (taps == 4) SP_TOK(V, 4);
    if (taps == 3) SP_TOK(V, 3);
    if (taps == 2) SP_TOK(V, 2);
    SP_TOK(V, 0);
  }
  SP_TOK(1, 0);
#undef SP_TOK
#undef SP_GO
}

// u: rows of the projection, x | B | C (`channels` columns) from column xbc_off, dt (heads columns) from dt_off;
// conv_w [channels][taps], the last column meets the current token; conv_state: the convolution's part of the requests'
// state rows.  xbc [tokens, channels]; dt, log_decay [tokens, heads] 32-bit.  `single`: every request has one token (a
// decode step); the convolution's memory is then moved on here, and `ullm_conv_state_update` is not needed.
extern "C" int ullm_ssd_prepare(int dtype, const void* u, long long row_stride, int xbc_off, int dt_off, int channels,
                                int heads, const void* conv_w, int taps, const float* conv_b, const float* dt_bias,
                                const float* a_log, float* conv_state, long long state_stride, int num_slots,
                                const int* cu_q, const int* token_req, const int* req_slots, int tokens, void* xbc,
                                float* dt, float* log_decay, int single, int* status, void* stream) {
  cudaStream_t st = (cudaStream_t)stream;
  if (tokens < 0 || channels <= 0 || heads <= 0 || taps < 1 || conv_b == nullptr || (taps > 1 && (conv_state == nullptr || num_slots <= 0)))
    return ULLM_ERR_BAD_SIZE;
  if (taps > SSD_MAX_TAPS) return ULLM_ERR_UNSUPPORTED;
  if (tokens == 0) return ULLM_OK;
#define SP_ARGS                                                                                                       \
  u, row_stride, xbc_off, dt_off, channels, heads, conv_w, taps, conv_b, dt_bias, a_log, conv_state, state_stride,    \
      num_slots, cu_q, token_req, req_slots, tokens, xbc, dt, log_decay, single, status, st
  if (dtype == ULLM_DTYPE_F32) return prepare_go<float>(SP_ARGS);
  if (dtype == ULLM_DTYPE_BF16) return prepare_go<__nv_bfloat16>(SP_ARGS);
  if (dtype == ULLM_DTYPE_F16) return prepare_go<__half>(SP_ARGS);
#undef SP_ARGS
  return ULLM_ERR_BAD_DTYPE;
}

template <typename T>
static int recurrence_go(const void* xbc, long long row_stride, int b_off, int c_off, const float* dt,
                         const float* log_decay, const float* d_skip, float* state, long long state_stride,
                         const int* cu_q, const int* req_slots, const int* token_req, float* out, int requests, int heads,
                         int n_state, int pdim, int groups, int num_slots, int most_tokens, int* status,
                         long long dt_stride, int silu_in, cudaStream_t st) {
  int rs = 1;  // lanes that share a column: as many as leave a thread about 8 rows, at most a warp
  while (rs < 32 && rs * 8 < n_state) rs <<= 1;
  const int col_groups = SSD_THREADS / rs;
  const int rows = (n_state + rs - 1) / rs;
  const int rpt = rows <= 4 ? 4 : (rows <= 8 ? 8 : 16);
  int sms = 148, dev = 0;
  if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  // columns per thread: time is (waves of blocks, two resident per SM) x (a token's cost, which grows slowly with them)
  int cpt = 1;
  if (rpt <= 8) {
    double best = 1e30;
    for (int c = 1; c <= 4; c *= 2) {
      const long long blocks = (long long)((pdim + c * col_groups - 1) / (c * col_groups)) * heads * requests;
      const double cost = (double)((blocks + 2LL * sms - 1) / (2LL * sms)) * (1.0 + 0.25 * (c - 1));
      if (cost < best - 1e-9) {
        best = cost;
        cpt = c;
      }
    }
  }
  const int cpb = col_groups * cpt, dimp = rpt * rs;
  const int per_tok = 2 * dimp + cpb + 4;
  int chunk = (40 * 1024 / 4) / (2 * per_tok);  // two buffers in at most 40 KB of shared memory
  chunk = chunk < 1 ? 1 : (chunk > 32 ? 32 : chunk);
  const size_t smem = (size_t)2 * chunk * per_tok * sizeof(float);
  const dim3 grid((pdim + cpb - 1) / cpb, heads, requests), block(2 * SSD_THREADS);
#define SSD_GO(RPT, CPT)                                                                                              \
  return ullm_launch_kernel(ssd_recurrence_kernel<T, RPT, CPT>, grid, block, smem, st, (const T*)xbc, row_stride, b_off, \
                            c_off, dt, log_decay, d_skip, state, state_stride, cu_q, req_slots, token_req, out, heads, \
                            n_state, pdim, heads / groups, rs, chunk, num_slots, most_tokens, status, dt_stride, silu_in)
  if (rpt == 4) {
    if (cpt == 4) SSD_GO(4, 4);
    if (cpt == 2) SSD_GO(4, 2);
    SSD_GO(4, 1);
  }
  if (rpt == 8) {
    if (cpt == 4) SSD_GO(8, 4);
    if (cpt == 2) SSD_GO(8, 2);
    SSD_GO(8, 1);
  }
  SSD_GO(16, 1);
#undef SSD_GO
}

// xbc [tokens, row_stride]: x in columns 0 .. heads * pdim - 1, B and C (groups * n_state each) from b_off and c_off.
// Requests that bring more than `most_tokens` tokens are left alone.  `dt_stride`: floats between two tokens' steps and
// decays (heads, or 0 for one row that serves all tokens); `silu_in`: x, B and C pass a silu as they are read.
extern "C" int ullm_ssd_recurrence(int dtype, const void* xbc, long long row_stride, int b_off, int c_off,
                                   const float* dt, const float* log_decay, const float* d_skip, float* state,
                                   long long state_stride, const int* cu_q, const int* req_slots, const int* token_req,
                                   float* out, int requests, int heads, int n_state, int pdim, int groups, int num_slots,
                                   int most_tokens, int* status, void* stream, long long dt_stride, int silu_in) {
  cudaStream_t st = (cudaStream_t)stream;
  if (requests < 0 || num_slots <= 0 || !ullm_ssd_supported(heads, n_state, pdim, groups, 1)) return ULLM_ERR_BAD_SIZE;
  if (requests > 65535) return ULLM_ERR_UNSUPPORTED;
  if (state_stride < (long long)heads * pdim * n_state) return ULLM_ERR_BAD_SIZE;
  if (requests == 0) return ULLM_OK;
#define SR_ARGS                                                                                                    \
  xbc, row_stride, b_off, c_off, dt, log_decay, d_skip, state, state_stride, cu_q, req_slots, token_req, out,      \
      requests, heads, n_state, pdim, groups, num_slots, most_tokens, status, dt_stride, silu_in, st
  if (dtype == ULLM_DTYPE_F32) return recurrence_go<float>(SR_ARGS);
  if (dtype == ULLM_DTYPE_BF16) return recurrence_go<__nv_bfloat16>(SR_ARGS);
  if (dtype == ULLM_DTYPE_F16) return recurrence_go<__half>(SR_ARGS);
#undef SR_ARGS
  return ULLM_ERR_BAD_DTYPE;
}

template <typename T>
static int gate_norm_go(const float* y, const void* z, long long z_stride, const float* w, void* out, int tokens,
                        int inner, int parts, float eps, int gate_behind, cudaStream_t st) {
  const int part = inner / parts;
  const size_t smem = (size_t)part * sizeof(float);
  if (smem > 160 * 1024) return ULLM_ERR_UNSUPPORTED;
  constexpr int V = 16 / (int)sizeof(T);
  const bool wide = part % V == 0 && z_stride % V == 0 &&
                    (((uintptr_t)y | (uintptr_t)z | (uintptr_t)w | (uintptr_t)out) & 15) == 0;
  int threads = 32;
  while (threads < 512 && threads * (wide ? V : 1) < part) threads <<= 1;
#define SG_GO(VEC)                                                                                                    \
  {                                                                                                                   \
    if (smem > 48 * 1024 && cudaFuncSetAttribute(ssd_gate_norm_kernel<T, VEC>,                                        \
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) { \
      cudaGetLastError();                                                                                             \
      return ULLM_ERR_LAUNCH;                                                                                         \
    }                                                                                                                 \
    return ullm_launch_kernel(ssd_gate_norm_kernel<T, VEC>, dim3(tokens, parts), dim3(threads), smem, st, y,          \
                              (const T*)z, z_stride, w, (T*)out, inner, part, eps, gate_behind);                                   \
  }
  if (wide) SG_GO(V);
  SG_GO(1);
#undef SG_GO
}

// out [tokens, inner] = norm of y * silu(z) over `parts` equal stretches, times w, or with `gate_behind` norm of y times w
// times sigmoid(z); y 32-bit, z rows z_stride apart.
extern "C" int ullm_ssd_gate_norm(int dtype, const float* y, const void* z, long long z_stride, const float* w, void* out,
                                  int tokens, int inner, int parts, float eps, void* stream, int gate_behind) {
  cudaStream_t st = (cudaStream_t)stream;
  if (tokens < 0 || inner <= 0 || parts <= 0 || inner % parts || parts > 65535 || z_stride < inner) return ULLM_ERR_BAD_SIZE;
  if (tokens == 0) return ULLM_OK;
  if (dtype == ULLM_DTYPE_F32) return gate_norm_go<float>(y, z, z_stride, w, out, tokens, inner, parts, eps, gate_behind, st);
  if (dtype == ULLM_DTYPE_BF16) return gate_norm_go<__nv_bfloat16>(y, z, z_stride, w, out, tokens, inner, parts, eps, gate_behind, st);
  if (dtype == ULLM_DTYPE_F16) return gate_norm_go<__half>(y, z, z_stride, w, out, tokens, inner, parts, eps, gate_behind, st);
  return ULLM_ERR_BAD_DTYPE;
}
