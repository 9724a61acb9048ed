// What lies between an attention's q | k | v projection and its scores, in its general form, for any mix of
// requests in one flat batch (prompt portions beside single decoded tokens):
//
//   1. optionally a short causal convolution over time on every channel of q, k and v:
//        y_t[c] = sum_j w[c][j] u_(t - taps + 1 + j)[c]
//      The taps - 1 projected rows that precede a step's first token come from the request's state row
//      ([taps - 1][row width] floats, zeros for a new request; row s holds the token taps - 1 - s places before
//      the step's first).  `conv_state_update` moves the state on after the step.
//   2. optionally a per-head RMS norm of q and k BEFORE the rotation, with or without a weight;
//   3. the rotation of the first `rotary_dim` dimensions of every q and k head, dimension i with dimension
//      i + rotary_dim / 2, by the angle position * inv_freq[i] (the 32-bit product; sincosf with full range
//      reduction: no table per position, no largest position);
//   4. optionally the unit RMS norm of q and k AFTER the rotation (no weight);
//   5. optionally value mixing across layers: the first layer that mixes leaves its values of the step's tokens
//      in `v_first`, every later one computes v <- (1 - lambda) v + lambda v_first;
//      optionally every query is multiplied by 1 + coef ln(floor((p + 1) / every) + 1) at position p;
//   6. k and v go to their cache slots, q to `q_out` [T, heads * head_dim].
//
// One warp per (token, head) over the q heads, the k heads and the v heads; rotation and stores alone (nothing of 1, 2, 4
// and 5) at sizes that allow 16-byte pieces run one block per token.  All arithmetic is 32-bit; a value is
// rounded once, when it is stored.
#include "common.cuh"

#define PREP_MAX_DIM 512
#define PREP_WARPS 4
#define PREP_MAX_TAPS 32

template <typename T>
__global__ void qkv_prepare_kernel(const T* __restrict__ qkv, long long row_stride, int tokens, int num_q, int num_kv,
                                   int head_dim, int v_dim, const T* __restrict__ conv_w, int taps,
                                   const float* __restrict__ conv_state, long long state_stride,
                                   const int* __restrict__ cu_q, const int* __restrict__ token_req,
                                   const int* __restrict__ req_slots, int num_state_slots,
                                   const int* __restrict__ positions, const float* __restrict__ inv_freq,
                                   int rotary_dim, const float* __restrict__ q_w, const float* __restrict__ k_w,
                                   int norm_first, int norm_last, float eps, int vmix_mode,
                                   const float* __restrict__ vmix_lambda, T* __restrict__ v_first,
                                   const int* __restrict__ slot_mapping, T* __restrict__ k_cache,
                                   T* __restrict__ v_cache, long long num_slots, T* __restrict__ q_out, int* status,
                                   float temp_coef, int temp_every) {
  __shared__ float buf[PREP_WARPS][PREP_MAX_DIM];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int units_per_token = num_q + 2 * num_kv;
  const long long unit = (long long)blockIdx.x * PREP_WARPS + warp;
  if (unit >= (long long)tokens * units_per_token) return;
  const int t = (int)(unit / units_per_token);
  const int u = (int)(unit - (long long)t * units_per_token);
  const int kind = u < num_q ? 0 : (u < num_q + num_kv ? 1 : 2);  // q, k, v
  const int head = kind == 0 ? u : (kind == 1 ? u - num_q : u - num_q - num_kv);
  const int dim = kind == 2 ? v_dim : head_dim;
  const int q_size = num_q * head_dim, k_size = num_kv * head_dim;
  const int chan0 = (kind == 0 ? 0 : (kind == 1 ? q_size : q_size + k_size)) + head * dim;  // column in the row
  const int r = token_req[t];
  float* x = buf[warp];

  // 1. the projected values, through the short convolution if there is one
  if (conv_w != nullptr && r >= 0) {
    const int t0 = cu_q[r];
    const int slot = req_slots[r];
    const bool slot_ok = taps > 1 && slot >= 0 && slot < num_state_slots;  // (one tap: no memory, no state row)
    if (taps > 1 && !slot_ok && lane == 0) ullm_report(status, ULLM_STATUS_SLOT, t, slot);
    const float* st = conv_state + (long long)(slot_ok ? slot : 0) * state_stride;
    const int row_width = q_size + k_size + num_kv * v_dim;
    for (int e = lane; e < dim; e += 32) {
      const int c = chan0 + e;
      float y = 0.f;
      for (int j = 0; j < taps; ++j) {
        const int back = taps - 1 - j;  // tokens before this one
        const int row = t - back;
        float uval;
        if (row >= t0) {
          uval = to_f32(qkv[(long long)row * row_stride + c]);
        } else {
          const int s = taps - 1 - (t0 - row);  // t0 - row in 1 .. taps - 1
          uval = slot_ok ? st[(long long)s * row_width + c] : 0.f;
        }
        y += to_f32(conv_w[(long long)c * taps + j]) * uval;
      }
      x[e] = y;
    }
  } else {
    for (int e = lane; e < dim; e += 32) x[e] = to_f32(qkv[(long long)t * row_stride + chan0 + e]);
  }
  __syncwarp();

  if (kind == 2) {
    // 5. value mixing, then the cache
    T* vf = v_first != nullptr ? v_first + (long long)t * num_kv * v_dim + head * v_dim : nullptr;
    const float lam = vmix_mode == 2 ? *vmix_lambda : 0.f;
    const int slot = slot_mapping != nullptr ? slot_mapping[t] : -1;
    const bool store = slot >= 0 && slot < num_slots;
    if (slot_mapping != nullptr && slot >= num_slots && lane == 0) ullm_report(status, ULLM_STATUS_SLOT, t, slot);
    T* dst = store ? v_cache + ((long long)slot * num_kv + head) * v_dim : nullptr;
    for (int e = lane; e < dim; e += 32) {
      float v = x[e];
      if (vmix_mode == 2) v = (1.f - lam) * v + lam * to_f32(vf[e]);
      const T rounded = from_f32<T>(v);
      if (vmix_mode == 1) vf[e] = rounded;
      if (store) dst[e] = rounded;
    }
    return;
  }

  const float* w = kind == 0 ? q_w : k_w;
  // 2. norm in front of the rotation
  if (norm_first) {
    float ss = 0.f;
    for (int e = lane; e < dim; e += 32) ss += x[e] * x[e];
    ss = warp_sum(ss);
    const float rstd = 1.f / sqrtf(ss / (float)dim + eps);
    for (int e = lane; e < dim; e += 32) x[e] = x[e] * rstd * (w != nullptr ? w[e] : 1.f);
    __syncwarp();
  }
  // 3. rotation
  if (rotary_dim > 0 && inv_freq != nullptr) {
    const float p = (float)positions[t];
    const int half = rotary_dim >> 1;
    for (int i = lane; i < half; i += 32) {
      float sn, cs;
      sincosf(p * inv_freq[i], &sn, &cs);
      const float a = x[i], b = x[i + half];
      x[i] = a * cs - b * sn;
      x[i + half] = b * cs + a * sn;
    }
    __syncwarp();
  }
  // 4. unit norm behind the rotation
  float mult = 1.f;
  if (norm_last) {
    float ss = 0.f;
    for (int e = lane; e < dim; e += 32) ss += x[e] * x[e];
    ss = warp_sum(ss);
    mult = 1.f / sqrtf(ss / (float)dim + eps);
  }
  // 6. stores
  if (kind == 0) {
    if (temp_every > 0) mult *= 1.f + temp_coef * logf((float)((positions[t] + 1) / temp_every + 1));
    T* dst = q_out + ((long long)t * num_q + head) * head_dim;
    for (int e = lane; e < dim; e += 32) dst[e] = from_f32<T>(x[e] * mult);
  } else {
    const int slot = slot_mapping != nullptr ? slot_mapping[t] : -1;
    if (slot_mapping != nullptr && slot >= num_slots && lane == 0) ullm_report(status, ULLM_STATUS_SLOT, t, slot);
    if (slot >= 0 && slot < num_slots) {
      T* dst = k_cache + ((long long)slot * num_kv + head) * head_dim;
      for (int e = lane; e < dim; e += 32) dst[e] = from_f32<T>(x[e] * mult);
    }
  }
}

// The usual case without convolution, norms and value mixing: rotation and stores alone.  One block per token: its sines
// and cosines are formed once, in shared memory, for all heads; a thread then moves 8 + 8 elements of a head's rotated part
// (dimensions i .. i + 7 and their partners) or 8 elements that only pass, in 16-byte pieces (`VEC` elements each).
template <typename T, int VEC>
__global__ void qkv_rotate_store_kernel(const T* __restrict__ qkv, long long row_stride, int num_q, int num_kv,
                                        int head_dim, int v_dim, const int* __restrict__ positions,
                                        const float* __restrict__ inv_freq, int rotary_dim,
                                        const int* __restrict__ slot_mapping, T* __restrict__ k_cache,
                                        T* __restrict__ v_cache, long long num_slots, T* __restrict__ q_out, int* status) {
  extern __shared__ __align__(16) float rot_sm[];  // [half] cosines, [half] sines
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int half = rotary_dim >> 1;
  if (half > 0) {
    const float p = (float)positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(p * inv_freq[i], &rot_sm[half + i], &rot_sm[i]);
  }
  const int slot = slot_mapping != nullptr ? slot_mapping[t] : -1;
  if (slot_mapping != nullptr && slot >= num_slots && threadIdx.x == 0) ullm_report(status, ULLM_STATUS_SLOT, t, slot);
  const bool store = slot >= 0 && slot < num_slots;
  __syncthreads();
  const int rot_items = half / VEC, per_head = rot_items + (head_dim - rotary_dim) / VEC, v_items = v_dim / VEC;
  const int qk_heads = num_q + num_kv;
  const int qk_total = qk_heads * per_head, total = qk_total + num_kv * v_items;
  const T* row = qkv + (long long)t * row_stride;
  for (int i = threadIdx.x; i < total; i += blockDim.x) {
    float a[VEC];
    if (i >= qk_total) {  // a value
      if (!store) continue;
      const int c = (i - qk_total) * VEC;
      load_vec<T, VEC>(row + qk_heads * head_dim + c, a);
      store_vec<T, VEC>(v_cache + (long long)slot * num_kv * v_dim + c, a);
      continue;
    }
    const int h = i / per_head, e = i - h * per_head;
    T* dst;
    if (h < num_q) {
      dst = q_out + ((long long)t * num_q + h) * head_dim;
    } else {
      if (!store) continue;
      dst = k_cache + ((long long)slot * num_kv + (h - num_q)) * head_dim;
    }
    const T* src = row + (long long)h * head_dim;
    if (e < rot_items) {
      const int d = e * VEC;
      float b[VEC], cs[VEC], sn[VEC], x[VEC];
      load_vec<T, VEC>(src + d, a);
      load_vec<T, VEC>(src + half + d, b);
      load_vec32<VEC>(rot_sm + d, cs);
      load_vec32<VEC>(rot_sm + half + d, sn);
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        x[j] = a[j] * cs[j] - b[j] * sn[j];
        b[j] = b[j] * cs[j] + a[j] * sn[j];
      }
      store_vec<T, VEC>(dst + d, x);
      store_vec<T, VEC>(dst + half + d, b);
    } else {
      const int d = rotary_dim + (e - rot_items) * VEC;
      load_vec<T, VEC>(src + d, a);
      store_vec<T, VEC>(dst + d, a);
    }
  }
}

// The convolution, the weighted norm per head and the stores alone (no rotation, norm behind it or value mixing), in 16-byte
// pieces.  One thread: VEC neighbouring channels of TOK tokens in a row; the filter and the rows in front wait in
// registers, so every projected row is read once (as in csrc/ssd.cu).  The lanes of a head (head_dim / VEC of them, a power
// of two) sum their squares by shuffles.  `single`: every request of the step has one token; the thread that convolves a
// channel is then the only reader of its memory and moves it on itself.
template <typename T, int VEC, int TAPS, int TOK>
__global__ void __launch_bounds__(128)
qkv_conv_prepare_kernel(const T* __restrict__ qkv, long long row_stride, int tokens, int num_q, int num_kv, int head_dim,
                        int v_dim, const T* __restrict__ conv_w, float* __restrict__ conv_state, long long state_stride,
                        const int* __restrict__ cu_q, const int* __restrict__ token_req, const int* __restrict__ req_slots,
                        int num_state_slots, const int* __restrict__ positions, const float* __restrict__ q_w,
                        const float* __restrict__ k_w, float eps, const int* __restrict__ slot_mapping,
                        T* __restrict__ k_cache, T* __restrict__ v_cache, long long num_slots, T* __restrict__ q_out,
                        int* status, float temp_coef, int temp_every, int single) {
  pdl_launch_dependents();
  pdl_wait();
  const int q_size = num_q * head_dim, k_size = num_kv * head_dim, width = q_size + k_size + num_kv * v_dim;
  const int raw = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  const bool live = raw < width;  // (every lane takes part in the shuffles)
  const int c0 = live ? raw : 0;
  const int kind = c0 < q_size ? 0 : (c0 < q_size + k_size ? 1 : 2);
  const int lph = head_dim / VEC;
  const int tok0 = blockIdx.y * TOK, tok1 = min(tokens, tok0 + TOK);
  float cur[TOK][VEC];
#pragma unroll
  for (int i = 0; i < TOK; ++i)
    if (tok0 + i < tok1) load_vec<T, VEC>(qkv + (long long)(tok0 + i) * row_stride + c0, cur[i]);
  float w[TAPS][VEC];  // flat: element i * TAPS + j is channel c0 + i's tap j
#pragma unroll
  for (int j = 0; j < TAPS; ++j) load_vec<T, VEC>(conv_w + (long long)c0 * TAPS + j * VEC, w[j]);
  float nw[VEC];
  if (kind < 2) load_vec32<VEC>((kind == 0 ? q_w : k_w) + (c0 - (kind == 0 ? 0 : q_size)) % head_dim, nw);
  float win[TAPS - 1][VEC];
  int prev = -1, t0 = 0;
  float* st = nullptr;
#pragma unroll
  for (int i = 0; i < TOK; ++i) {
    const int t = tok0 + i;
    if (t >= tok1) break;
    const int r = token_req[t];
    float y[VEC];
    if (r < 0) {  // a row that belongs to no request: as projected (nothing reads it)
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = cur[i][e];
      prev = -1;
    } else {
      const bool fresh = r != prev;
      if (fresh) {
        prev = r;
        t0 = cu_q[r];
        const int slot = req_slots[r];
        st = nullptr;
        if (slot >= 0 && slot < num_state_slots) st = conv_state + (long long)slot * state_stride + c0;
        else ullm_report(status, ULLM_STATUS_SLOT, t, slot);
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
          const int back = TAPS - 1 - j;
          if (t - back >= t0) {
            load_vec<T, VEC>(qkv + (long long)(t - back) * row_stride + c0, win[j]);
          } else if (st != nullptr) {
            load_vec32<VEC>(st + (long long)(TAPS - 1 - (t0 - (t - back))) * width, win[j]);
          } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) win[j][e] = 0.f;
          }
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          const int f = e * TAPS + j;
          y[e] = fmaf(w[f / VEC][f % VEC], j < TAPS - 1 ? win[j < TAPS - 1 ? j : 0][e] : cur[i][e], y[e]);
        }
#pragma unroll
      for (int j = 0; j + 1 < TAPS - 1; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) win[j][e] = win[j + 1][e];
#pragma unroll
      for (int e = 0; e < VEC; ++e) win[TAPS - 2][e] = cur[i][e];
      if (single && live && st != nullptr) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) store_vec32<VEC>(st + (long long)j * width, win[j]);
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += y[e] * y[e];
    for (int d = lph >> 1; d > 0; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
    if (kind < 2) {
      float mult = 1.f / sqrtf(ss / (float)head_dim + eps);
      if (kind == 0 && temp_every > 0) mult *= 1.f + temp_coef * logf((float)((positions[t] + 1) / temp_every + 1));
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] *= mult * nw[e];
    }
    if (!live) continue;
    if (kind == 0) {
      store_vec<T, VEC>(q_out + (long long)t * q_size + c0, y);
    } else {
      const int slot = slot_mapping != nullptr ? slot_mapping[t] : -1;
      if (slot >= num_slots) ullm_report(status, ULLM_STATUS_SLOT, t, slot);
      if (slot >= 0 && slot < num_slots) {
        if (kind == 1) store_vec<T, VEC>(k_cache + (long long)slot * k_size + (c0 - q_size), y);
        else store_vec<T, VEC>(v_cache + (long long)slot * num_kv * v_dim + (c0 - q_size - k_size), y);
      }
    }
  }
}

// After a step: the state row of every request of the step holds the last taps - 1 projected rows.  One thread
// per (request, channel); rows are moved in ascending order, so a request that brought fewer than taps - 1 tokens
// shifts its old rows down before it appends (row s takes old row s + n: always a row not yet written).
template <typename T>
__global__ void conv_state_update_kernel(const T* __restrict__ qkv, long long row_stride, int row_width, int taps,
                                         float* __restrict__ conv_state, long long state_stride,
                                         const int* __restrict__ cu_q, const int* __restrict__ token_req,
                                         const int* __restrict__ req_slots, int num_state_slots, int requests) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.y;
  if (r >= requests) return;
  const int t0 = cu_q[r], t1 = cu_q[r + 1];
  const int n = t1 - t0;
  if (n <= 0 || token_req[t0] < 0) return;  // a padding row belongs to no request
  const int slot = req_slots[r];
  if (slot < 0 || slot >= num_state_slots) return;
  float* st = conv_state + (long long)slot * state_stride;
  for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < row_width; c += gridDim.x * blockDim.x) {
    for (int s = 0; s < taps - 1; ++s) {
      const int back = taps - 1 - s;  // rows before the end
      float v;
      if (back <= n) v = to_f32(qkv[(long long)(t1 - back) * row_stride + c]);
      else v = st[(long long)(s + n) * row_width + c];
      st[(long long)s * row_width + c] = v;
    }
  }
}

template <typename T>
static int prepare_launch(const void* qkv, long long row_stride, int tokens, int num_q, int num_kv, int head_dim,
                          int v_dim, const void* conv_w, int taps, const float* conv_state, long long state_stride,
                          const int* cu_q, const int* token_req, const int* req_slots, int num_state_slots,
                          const int* positions, const float* inv_freq, int rotary_dim, const float* q_w,
                          const float* k_w, int norm_first, int norm_last, float eps, int vmix_mode,
                          const float* vmix_lambda, void* v_first, const int* slot_mapping, void* k_cache,
                          void* v_cache, long long num_slots, void* q_out, int* status, float temp_coef, int temp_every,
                          cudaStream_t st) {
  constexpr int V = 16 / (int)sizeof(T);
  const bool plain = conv_w == nullptr && !norm_first && !norm_last && vmix_mode == 0 && temp_every <= 0 && head_dim % V == 0 &&
                     v_dim % V == 0 && rotary_dim % (2 * V) == 0 && row_stride % V == 0 &&
                     (((uintptr_t)qkv | (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) == 0;
  if (plain) {
    const int rot = inv_freq != nullptr ? rotary_dim : 0;
    const int items = (num_q + num_kv) * (head_dim - rot / 2) / V + num_kv * v_dim / V;
    int threads = 64;
    while (threads < 256 && threads < items) threads <<= 1;
    return ullm_launch_kernel(qkv_rotate_store_kernel<T, V>, dim3(tokens), dim3(threads), (size_t)rot * sizeof(float), st,
                              (const T*)qkv, row_stride, num_q, num_kv, head_dim, v_dim, positions, inv_freq, rot,
                              slot_mapping, (T*)k_cache, (T*)v_cache, num_slots, (T*)q_out, status);
  }
  const long long units = (long long)tokens * (num_q + 2 * num_kv);
  const long long blocks = (units + PREP_WARPS - 1) / PREP_WARPS;
  if (blocks > 0x7fffffffLL) return ULLM_ERR_BAD_SIZE;
  return ullm_launch_kernel(qkv_prepare_kernel<T>, dim3((int)blocks), dim3(PREP_WARPS * 32), 0, st, (const T*)qkv,
                            row_stride, tokens, num_q, num_kv, head_dim, v_dim, (const T*)conv_w, taps, conv_state,
                            state_stride, cu_q, token_req, req_slots, num_state_slots, positions, inv_freq, rotary_dim,
                            q_w, k_w, norm_first, norm_last, eps, vmix_mode, vmix_lambda, (T*)v_first, slot_mapping,
                            (T*)k_cache, (T*)v_cache, num_slots, (T*)q_out, status, temp_coef, temp_every);
}

// `temp_every` > 0: the queries' temperature (with `positions`), 0: none.
// `conv_w`: [row width][taps] in the engine's dtype (the q, k and v filters one after the other) or null.
// `vmix_mode`: 0 none, 1 this layer leaves its values in `v_first`, 2 it mixes them in with *vmix_lambda.
extern "C" int ullm_qkv_prepare(int dtype, const void* qkv, long long row_stride, int tokens, int num_q, int num_kv,
                                int head_dim, int v_dim, const void* conv_w, int taps, const float* conv_state,
                                long long state_stride, const int* cu_q, const int* token_req, const int* req_slots,
                                int num_state_slots, const int* positions, const float* inv_freq, int rotary_dim,
                                const float* q_w, const float* k_w, int norm_first, int norm_last, float eps,
                                int vmix_mode, const float* vmix_lambda, void* v_first, const int* slot_mapping,
                                void* k_cache, void* v_cache, long long num_slots, void* q_out, int* status,
                                void* stream, float temp_coef, int temp_every) {
  cudaStream_t st = (cudaStream_t)stream;
  if (tokens < 0 || num_q <= 0 || num_kv <= 0 || head_dim <= 0 || v_dim <= 0) return ULLM_ERR_BAD_SIZE;
  if (head_dim > PREP_MAX_DIM || v_dim > PREP_MAX_DIM || rotary_dim < 0 || rotary_dim > head_dim || (rotary_dim & 1))
    return ULLM_ERR_UNSUPPORTED;
  if (conv_w != nullptr && (taps < 1 || taps > PREP_MAX_TAPS || (taps > 1 && conv_state == nullptr)))
    return ULLM_ERR_UNSUPPORTED;
  if (vmix_mode < 0 || vmix_mode > 2 || (vmix_mode != 0 && v_first == nullptr) ||
      (vmix_mode == 2 && vmix_lambda == nullptr))
    return ULLM_ERR_BAD_SIZE;
  if (temp_every > 0 && positions == nullptr) return ULLM_ERR_BAD_SIZE;
  if (rotary_dim > 0 && (inv_freq == nullptr || positions == nullptr)) return ULLM_ERR_BAD_SIZE;
  if (tokens == 0) return ULLM_OK;
#define PREP_ARGS                                                                                                   \
  qkv, row_stride, tokens, num_q, num_kv, head_dim, v_dim, conv_w, taps, conv_state, state_stride, cu_q, token_req,  \
      req_slots, num_state_slots, positions, inv_freq, rotary_dim, q_w, k_w, norm_first, norm_last, eps, vmix_mode, \
      vmix_lambda, v_first, slot_mapping, k_cache, v_cache, num_slots, q_out, status, temp_coef, temp_every, st
  if (dtype == ULLM_DTYPE_F32) return prepare_launch<float>(PREP_ARGS);
  if (dtype == ULLM_DTYPE_BF16) return prepare_launch<__nv_bfloat16>(PREP_ARGS);
  if (dtype == ULLM_DTYPE_F16) return prepare_launch<__half>(PREP_ARGS);
#undef PREP_ARGS
  return ULLM_ERR_BAD_DTYPE;
}

extern "C" int ullm_conv_state_update(int dtype, const void* qkv, long long row_stride, int row_width, int taps,
                                      float* conv_state, long long state_stride, const int* cu_q,
                                      const int* token_req, const int* req_slots, int num_state_slots, int requests,
                                      void* stream) {
  cudaStream_t st = (cudaStream_t)stream;
  if (requests < 0 || row_width <= 0 || taps < 1 || taps > PREP_MAX_TAPS) return ULLM_ERR_BAD_SIZE;
  if (requests == 0 || taps == 1) return ULLM_OK;
  if (requests > 65535) return ULLM_ERR_UNSUPPORTED;
  const dim3 grid((row_width + 127) / 128, requests), block(128);
  if (dtype == ULLM_DTYPE_F32)
    return ullm_launch_kernel(conv_state_update_kernel<float>, grid, block, 0, st, (const float*)qkv, row_stride,
                              row_width, taps, conv_state, state_stride, cu_q, token_req, req_slots, num_state_slots,
                              requests);
  if (dtype == ULLM_DTYPE_BF16)
    return ullm_launch_kernel(conv_state_update_kernel<__nv_bfloat16>, grid, block, 0, st, (const __nv_bfloat16*)qkv,
                              row_stride, row_width, taps, conv_state, state_stride, cu_q, token_req, req_slots,
                              num_state_slots, requests);
  if (dtype == ULLM_DTYPE_F16)
    return ullm_launch_kernel(conv_state_update_kernel<__half>, grid, block, 0, st, (const __half*)qkv, row_stride,
                              row_width, taps, conv_state, state_stride, cu_q, token_req, req_slots, num_state_slots,
                              requests);
  return ULLM_ERR_BAD_DTYPE;
}

template <typename T>
static int conv_prepare_go(const void* qkv, long long row_stride, int tokens, int num_q, int num_kv, int head_dim, int v_dim,
                           const void* conv_w, int taps, float* conv_state, long long state_stride, const int* cu_q,
                           const int* token_req, const int* req_slots, int num_state_slots, const int* positions,
                           const float* q_w, const float* k_w, float eps, const int* slot_mapping, void* k_cache,
                           void* v_cache, long long num_slots, void* q_out, int* status, float temp_coef, int temp_every,
                           int single, cudaStream_t st) {
  constexpr int V = 16 / (int)sizeof(T);
  const int lph = head_dim / V;
  if (head_dim % V || v_dim % V || lph > 32 || (lph & (lph - 1)) || row_stride % V || state_stride % 4 ||
      (((uintptr_t)qkv | (uintptr_t)conv_w | (uintptr_t)conv_state | (uintptr_t)q_w | (uintptr_t)k_w | (uintptr_t)k_cache |
        (uintptr_t)v_cache | (uintptr_t)q_out) & 15))
    return ULLM_ERR_UNSUPPORTED;
  const int width = num_q * head_dim + num_kv * (head_dim + v_dim);
  const int tok = tokens >= 512 ? 4 : 1, threads = 128;
  const dim3 grid((width / V + threads - 1) / threads, (tokens + tok - 1) / tok), block(threads);
  if (grid.y > 65535) return ULLM_ERR_UNSUPPORTED;
#define CP_AS(TAPS, TOK)                                                                                              \
  return ullm_launch_kernel(qkv_conv_prepare_kernel<T, V, TAPS, TOK>, grid, block, 0, st, (const T*)qkv, row_stride,  \
                            tokens, num_q, num_kv, head_dim, v_dim, (const T*)conv_w, conv_state, state_stride, cu_q, \
                            token_req, req_slots, num_state_slots, positions, q_w, k_w, eps, slot_mapping,            \
                            (T*)k_cache, (T*)v_cache, num_slots, (T*)q_out, status, temp_coef, temp_every, single)
#define CP_GO(TAPS)              \
  {                              \
    if (tok == 4) CP_AS(TAPS, 4); \
    CP_AS(TAPS, 1);              \
  }
  if (taps == 2) CP_GO(2);
  if (taps == 3) CP_GO(3);
  if (taps == 4) CP_GO(4);
#undef CP_GO
#undef CP_AS
  return ULLM_ERR_UNSUPPORTED;
}

// `ullm_qkv_prepare` for a convolution of 2 to 4 taps and weighted norms per head without a rotation, in 16-byte pieces;
// with `single` (every request of the step has one token) the convolution's memory is moved on here and
// `ullm_conv_state_update` is not needed.  ULLM_ERR_UNSUPPORTED (nothing has run): other sizes or alignments.
extern "C" int ullm_qkv_conv_prepare(int dtype, const void* qkv, long long row_stride, int tokens, int num_q, int num_kv,
                                     int head_dim, int v_dim, const void* conv_w, int taps, float* conv_state,
                                     long long state_stride, const int* cu_q, const int* token_req, const int* req_slots,
                                     int num_state_slots, const int* positions, const float* q_w, const float* k_w, float eps,
                                     const int* slot_mapping, void* k_cache, void* v_cache, long long num_slots, void* q_out,
                                     int* status, float temp_coef, int temp_every, int single, void* stream) {
  cudaStream_t st = (cudaStream_t)stream;
  if (tokens < 0 || num_q <= 0 || num_kv <= 0 || head_dim <= 0 || v_dim <= 0) return ULLM_ERR_BAD_SIZE;
  if (conv_w == nullptr || conv_state == nullptr || q_w == nullptr || k_w == nullptr || (temp_every > 0 && positions == nullptr))
    return ULLM_ERR_UNSUPPORTED;
  if (tokens == 0) return ULLM_OK;
#define CP_ARGS                                                                                                       \
  qkv, row_stride, tokens, num_q, num_kv, head_dim, v_dim, conv_w, taps, conv_state, state_stride, cu_q, token_req,    \
      req_slots, num_state_slots, positions, q_w, k_w, eps, slot_mapping, k_cache, v_cache, num_slots, q_out, status, \
      temp_coef, temp_every, single, st
  if (dtype == ULLM_DTYPE_F32) return conv_prepare_go<float>(CP_ARGS);
  if (dtype == ULLM_DTYPE_BF16) return conv_prepare_go<__nv_bfloat16>(CP_ARGS);
  if (dtype == ULLM_DTYPE_F16) return conv_prepare_go<__half>(CP_ARGS);
#undef CP_ARGS
  return ULLM_ERR_BAD_DTYPE;
}
