// Row kernels of a 32-bit residual stream whose sub-layers are normed on BOTH sides
// (x <- x + norm_b(f(norm_a(x)))), with norms that may subtract the mean:
//
//   norm_add_norm   stream[t] += mult * w * n(a[t])            (a absent: nothing is added)
//                   stream[t] += extra_rows[t]; stream[t] += extra_vec     (each optional, in this order)
//                   out[t] = round(w2 * n2(stream[t]))          (optional: the norm that reads the stream next)
//   norm_rows       out[r] = round(w * n(stream[rows[r]]))      (gathered rows; `rows` null: all in order)
//   pair_norm_add_norm   stream[t] += mult * (wa * n(a[t]) + wb * n(b[t])) for TWO sub-layers' outputs, each divided by
//                   its own root mean square; then out as above.  Without a stream: rows_out[t] = round(the sum)
//                   With an outer norm: stream[t] += mult_o * wo * n(s) for s = the sum of the two
//   relu2           out = round(max(in, 0)^2)
//   act_rows        out = round(act(in)) on a column range of wider rows: silu or the exact gelu
//   xielu           out = round(act(in)), act(z) = softplus(p) z^2 + z / 2 for z > 0,
//                                          (1/2 + softplus(q)) (e^z - 1 - z) + z / 2 otherwise
//
// n(v) = v / sqrt(mean(v^2) + eps), or with `center` = 1 (v - mean(v)) / sqrt(mean((v - mean(v))^2) + eps): the
// variance is the mean of the squared deviations, formed in a second pass over the row, which waits in shared
// memory.  The norm that reads the stream next may also be `center2` = 2, a norm without statistics:
// out = tanh(alpha * s) * w2 + b2 with one number alpha and a vector b2, or `center2` = 3, no norm at all: out is the
// stream rounded.  `center` = 2 for the added operand: n(v) = v, so stream[t] += mult * w * a[t] (a scale per channel on a
// sub-layer's output; w null: no scale), the arrangement of a pre-norm layer on a 32-bit stream.  Sums, means and the stream are 32-bit; one rounding at each store.  One block per row.
#include "common.cuh"

#define SN_MAX_SMEM (160 * 1024)

// (sum of v, then sum of squared deviations) or (sum of squares): returns the factor 1 / sqrt(.. + eps) and
// leaves the mean (0 without `center`) in *mean_out.
__device__ __forceinline__ float row_rstd(const float* row, int cols, bool center, float eps, float* scratch,
                                          float* mean_out) {
  float mean = 0.f;
  if (center) {
    float acc = 0.f;
    for (int c = threadIdx.x; c < cols; c += blockDim.x) acc += row[c];
    mean = block_sum(acc, scratch) / (float)cols;
  }
  float acc = 0.f;
  for (int c = threadIdx.x; c < cols; c += blockDim.x) {
    const float d = row[c] - mean;
    acc += d * d;
  }
  *mean_out = mean;
  return 1.f / sqrtf(block_sum(acc, scratch) / (float)cols + eps);
}

template <typename TA, typename TO>
__global__ void norm_add_norm_kernel(const TA* __restrict__ a, float* __restrict__ stream,
                                     const float* __restrict__ w, int cols, float eps, float mult, int center,
                                     const float* __restrict__ extra_rows, const float* __restrict__ extra_vec,
                                     const float* __restrict__ w2, float eps2, int center2, TO* __restrict__ out,
                                     const float* __restrict__ alpha2, const float* __restrict__ b2) {
  extern __shared__ float sn_smem[];  // [cols] the operand's row, then [cols] the stream's row
  __shared__ float scratch[33];
  pdl_launch_dependents();
  pdl_wait();
  const long long base = (long long)blockIdx.x * cols;
  float* row_a = sn_smem;
  float* row_s = sn_smem + cols;
  float rstd = 0.f, mean = 0.f;
  if (a != nullptr) {
    for (int c = threadIdx.x; c < cols; c += blockDim.x) row_a[c] = to_f32(a[base + c]);
    __syncthreads();
    rstd = 1.f;
    if (center != 2) rstd = row_rstd(row_a, cols, center != 0, eps, scratch, &mean);
  }
  for (int c = threadIdx.x; c < cols; c += blockDim.x) {
    float s = stream[base + c];
    if (a != nullptr) s += mult * ((row_a[c] - mean) * rstd * (w != nullptr ? w[c] : 1.f));
    if (extra_rows != nullptr) s += extra_rows[base + c];
    if (extra_vec != nullptr) s += extra_vec[c];
    stream[base + c] = s;
    if (center2 == 3) {
      if (out != nullptr) out[base + c] = from_f32<TO>(s);
    } else {
      row_s[c] = s;
    }
  }
  if (out == nullptr || center2 == 3) return;
  if (center2 == 2) {  // (a thread reads what it wrote itself: no barrier)
    const float al = *alpha2;
    for (int c = threadIdx.x; c < cols; c += blockDim.x)
      out[base + c] = from_f32<TO>(tanhf(al * row_s[c]) * w2[c] + b2[c]);
    return;
  }
  __syncthreads();
  float mean2;
  const float rstd2 = row_rstd(row_s, cols, center2 != 0, eps2, scratch, &mean2);
  for (int c = threadIdx.x; c < cols; c += blockDim.x)
    out[base + c] = from_f32<TO>((row_s[c] - mean2) * rstd2 * w2[c]);
}

// Two sub-layers' rows a and b, each divided by its own root mean square and weighted, their sum (times `mult`) added
// to the stream; then the norm that reads the stream next.  One block per row; VEC neighbouring columns per thread and
// turn (16-byte pieces where the rows allow), both sums of squares in one set of barriers.
template <typename T, int VEC>
__global__ void pair_norm_add_norm_kernel(const T* __restrict__ a, const T* __restrict__ b,
                                          const float* __restrict__ wa, const float* __restrict__ wb, int cols,
                                          float eps, float mult, float* __restrict__ stream, T* __restrict__ rows_out,
                                          const float* __restrict__ w2, float eps2, int kind2,
                                          const float* __restrict__ alpha2, const float* __restrict__ b2,
                                          T* __restrict__ out, const float* __restrict__ wo, float eps_o, float mult_o) {
  extern __shared__ __align__(16) float sn_smem[];  // [cols] a, [cols] b; the stream's row takes a's place
  __shared__ float sums[2][33];
  pdl_launch_dependents();
  pdl_wait();
  const long long base = (long long)blockIdx.x * cols;
  float* row_a = sn_smem;
  float* row_b = sn_smem + cols;
  float qa = 0.f, qb = 0.f;
  for (int c0 = threadIdx.x * VEC; c0 < cols; c0 += blockDim.x * VEC) {
    float va[VEC], vb[VEC];
    load_vec<T, VEC>(a + base + c0, va);
    load_vec<T, VEC>(b + base + c0, vb);
    store_vec32<VEC>(row_a + c0, va);
    store_vec32<VEC>(row_b + c0, vb);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      qa += va[i] * va[i];
      qb += vb[i] * vb[i];
    }
  }
  qa = warp_sum(qa);
  qb = warp_sum(qb);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
  if (lane == 0) {
    sums[0][warp] = qa;
    sums[1][warp] = qb;
  }
  __syncthreads();
  qa = qb = 0.f;
  for (int i = 0; i < nwarps; ++i) {  // (every thread adds the warps' sums in the same order)
    qa += sums[0][i];
    qb += sums[1][i];
  }
  const float ra = mult / sqrtf(qa / (float)cols + eps), rb = mult / sqrtf(qb / (float)cols + eps);
  float ro = 1.f;
  if (wo != nullptr) {  // the weighted sum takes b's place and is normed as one row
    float qo = 0.f;
    for (int c0 = threadIdx.x * VEC; c0 < cols; c0 += blockDim.x * VEC) {
      float ga[VEC], gb[VEC], va[VEC], vb[VEC];
      load_vec32<VEC>(wa + c0, ga);
      load_vec32<VEC>(wb + c0, gb);
      load_vec32<VEC>(row_a + c0, va);
      load_vec32<VEC>(row_b + c0, vb);
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        vb[i] = va[i] * ra * ga[i] + vb[i] * rb * gb[i];
        qo += vb[i] * vb[i];
      }
      store_vec32<VEC>(row_b + c0, vb);
    }
    qo = warp_sum(qo);
    __syncthreads();  // the two sums have been read
    if (lane == 0) sums[0][warp] = qo;
    __syncthreads();
    qo = 0.f;
    for (int i = 0; i < nwarps; ++i) qo += sums[0][i];
    ro = mult_o / sqrtf(qo / (float)cols + eps_o);
  }
  const float al = (out != nullptr && kind2 == 2) ? *alpha2 : 0.f;
  for (int c0 = threadIdx.x * VEC; c0 < cols; c0 += blockDim.x * VEC) {
    float s[VEC];
    if (stream != nullptr) load_vec32<VEC>(stream + base + c0, s);
    else
#pragma unroll
      for (int i = 0; i < VEC; ++i) s[i] = 0.f;
    float ga[VEC], gb[VEC], va[VEC], vb[VEC];
    load_vec32<VEC>(row_b + c0, vb);
    if (wo != nullptr) {
      load_vec32<VEC>(wo + c0, ga);
#pragma unroll
      for (int i = 0; i < VEC; ++i) s[i] += vb[i] * ro * ga[i];
    } else {
      load_vec32<VEC>(row_a + c0, va);
      load_vec32<VEC>(wa + c0, ga);
      load_vec32<VEC>(wb + c0, gb);
#pragma unroll
      for (int i = 0; i < VEC; ++i) s[i] += va[i] * ra * ga[i] + vb[i] * rb * gb[i];
    }
    if (stream != nullptr) store_vec32<VEC>(stream + base + c0, s);
    if (rows_out != nullptr) store_vec<T, VEC>(rows_out + base + c0, s);
    if (out == nullptr) continue;
    if (kind2 == 3) {
      store_vec<T, VEC>(out + base + c0, s);
    } else if (kind2 == 2) {
      float g2[VEC], d2[VEC];
      load_vec32<VEC>(w2 + c0, g2);
      load_vec32<VEC>(b2 + c0, d2);
#pragma unroll
      for (int i = 0; i < VEC; ++i) s[i] = tanhf(al * s[i]) * g2[i] + d2[i];
      store_vec<T, VEC>(out + base + c0, s);
    } else {
      store_vec32<VEC>(row_a + c0, s);
    }
  }
  if (out == nullptr || kind2 >= 2) return;
  __syncthreads();
  float mean2;
  const float rstd2 = row_rstd(row_a, cols, kind2 != 0, eps2, sums[0], &mean2);
  for (int c = threadIdx.x; c < cols; c += blockDim.x)
    out[base + c] = from_f32<T>((row_a[c] - mean2) * rstd2 * w2[c]);
}

template <typename TO>
__global__ void norm_rows_kernel(const float* __restrict__ stream, const int* __restrict__ rows,
                                 const float* __restrict__ w, TO* __restrict__ out, int cols, int src_rows, float eps,
                                 int center, int* status, const float* __restrict__ alpha,
                                 const float* __restrict__ b) {
  extern __shared__ float sn_smem[];
  __shared__ float scratch[33];
  pdl_launch_dependents();
  pdl_wait();
  int r = rows != nullptr ? rows[blockIdx.x] : (int)blockIdx.x;
  const bool bad = r < 0 || r >= src_rows;
  if (bad) {
    if (threadIdx.x == 0) ullm_report(status, ULLM_STATUS_ROW, blockIdx.x, r);
    r = 0;
  }
  const float* s = stream + (long long)r * cols;
  if (center == 2) {
    const float al = *alpha;
    for (int c = threadIdx.x; c < cols; c += blockDim.x)
      out[(long long)blockIdx.x * cols + c] = from_f32<TO>(bad ? 0.f : tanhf(al * s[c]) * w[c] + b[c]);
    return;
  }
  for (int c = threadIdx.x; c < cols; c += blockDim.x) sn_smem[c] = s[c];
  __syncthreads();
  float mean;
  const float rstd = row_rstd(sn_smem, cols, center != 0, eps, scratch, &mean);
  for (int c = threadIdx.x; c < cols; c += blockDim.x)
    out[(long long)blockIdx.x * cols + c] = from_f32<TO>(bad ? 0.f : (sn_smem[c] - mean) * rstd * w[c]);
}

__device__ __forceinline__ float softplus_f32(float v) { return log1pf(expf(-fabsf(v))) + fmaxf(v, 0.f); }

template <typename T>
__global__ void xielu_kernel(const T* __restrict__ in, T* __restrict__ out, long long n,
                             const float* __restrict__ pq) {
  pdl_launch_dependents();
  pdl_wait();
  const float ap = softplus_f32(pq[0]), aq = 0.5f + softplus_f32(pq[1]);
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const float z = to_f32(in[i]);
    const float y = z > 0.f ? ap * z * z + 0.5f * z : aq * (expm1f(z) - z) + 0.5f * z;
    out[i] = from_f32<T>(y);
  }
}

// out = max(in, 0)^2, VEC elements per thread and turn
template <typename T, int VEC>
__global__ void relu2_kernel(const T* in, T* out, long long n) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * VEC; i < n;
       i += (long long)gridDim.x * blockDim.x * VEC) {
    float v[VEC];
    load_vec<T, VEC>(in + i, v);
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
      const float r = fmaxf(v[k], 0.f);
      v[k] = r * r;
    }
    store_vec<T, VEC>(out + i, v);
  }
}

// out[r][c] = act(in[r][c]) for a column range of wider rows (strides in elements; `out` may be `in`): ACT 0 silu,
// 1 the exact gelu z (1 + erf(z / sqrt 2)) / 2
template <typename T, int VEC, int ACT>
__global__ void act_rows_kernel(const T* in, long long in_stride, T* out, long long out_stride, long long pieces,
                                int per_row) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < pieces; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / per_row;
    const int c = (int)(i - r * per_row) * VEC;
    float v[VEC];
    load_vec<T, VEC>(in + r * in_stride + c, v);
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = ACT == 0 ? act_silu(v[k]) : 0.5f * v[k] * (1.f + erff(v[k] * 0.70710678118654752f));
    store_vec<T, VEC>(out + r * out_stride + c, v);
  }
}

static inline int sn_threads(int cols) {
  int threads = 32;
  while (threads < 512 && threads * 4 < cols) threads <<= 1;
  return threads;
}

template <typename K>
static int sn_allow_smem(K kernel, size_t smem) {
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return ULLM_ERR_UNSUPPORTED;
  }
  return ULLM_OK;
}

template <typename TA, typename TO>
static int norm_add_norm_launch(const void* a, float* stream, const float* w, int rows, int cols, float eps,
                                float mult, int center, const float* extra_rows, const float* extra_vec,
                                const float* w2, float eps2, int center2, void* out, const float* alpha2,
                                const float* b2, cudaStream_t st) {
  const size_t smem = 2 * (size_t)cols * sizeof(float);
  if (smem > SN_MAX_SMEM) return ULLM_ERR_UNSUPPORTED;
  const int rc = sn_allow_smem(norm_add_norm_kernel<TA, TO>, smem);
  if (rc != ULLM_OK) return rc;
  return ullm_launch_kernel(norm_add_norm_kernel<TA, TO>, dim3(rows), dim3(sn_threads(cols)), smem, st,
                            (const TA*)a, stream, w, cols, eps, mult, center, extra_rows, extra_vec, w2, eps2,
                            center2, (TO*)out, alpha2, b2);
}

// `a_dtype`: dtype of `a` (the engine's, or 32-bit for a sub-layer that leaves 32-bit rows); `out_dtype`: of `out`.
// `a` null: nothing is normed and added (then `w` is unused); `out` null: no next norm.
extern "C" int ullm_norm_add_norm(int a_dtype, const void* a, float* stream, const float* w, int rows, int cols,
                                  float eps, float mult, int center, const float* extra_rows,
                                  const float* extra_vec, const float* w2, float eps2, int center2, int out_dtype,
                                  void* out, void* stream_handle, const float* alpha2, const float* b2) {
  cudaStream_t st = (cudaStream_t)stream_handle;
  if (rows < 0 || cols <= 0) return ULLM_ERR_BAD_SIZE;
  if ((a != nullptr && w == nullptr && center != 2) || (out != nullptr && w2 == nullptr && center2 != 3)) return ULLM_ERR_BAD_SIZE;
  if (center < 0 || center > 2 || center2 < 0 || center2 > 3) return ULLM_ERR_BAD_SIZE;
  if (out != nullptr && center2 == 2 && (alpha2 == nullptr || b2 == nullptr)) return ULLM_ERR_BAD_SIZE;
  if (rows == 0) return ULLM_OK;
#define SN_GO(TA, TO)                                                                                              \
  return norm_add_norm_launch<TA, TO>(a, stream, w, rows, cols, eps, mult, center, extra_rows, extra_vec, w2, eps2, \
                                      center2, out, alpha2, b2, st)
#define SN_OUT(TA)                                         \
  if (out_dtype == ULLM_DTYPE_F32) SN_GO(TA, float);       \
  if (out_dtype == ULLM_DTYPE_BF16) SN_GO(TA, __nv_bfloat16); \
  if (out_dtype == ULLM_DTYPE_F16) SN_GO(TA, __half);      \
  return ULLM_ERR_BAD_DTYPE
  if (a_dtype == ULLM_DTYPE_F32) { SN_OUT(float); }
  if (a_dtype == ULLM_DTYPE_BF16) { SN_OUT(__nv_bfloat16); }
  if (a_dtype == ULLM_DTYPE_F16) { SN_OUT(__half); }
#undef SN_OUT
#undef SN_GO
  return ULLM_ERR_BAD_DTYPE;
}

template <typename TO>
static int norm_rows_launch(const float* stream, const int* rows, const float* w, void* out, int count, int cols,
                            int src_rows, float eps, int center, int* status, const float* alpha, const float* b,
                            cudaStream_t st) {
  const size_t smem = (size_t)cols * sizeof(float);
  if (smem > SN_MAX_SMEM) return ULLM_ERR_UNSUPPORTED;
  const int rc = sn_allow_smem(norm_rows_kernel<TO>, smem);
  if (rc != ULLM_OK) return rc;
  return ullm_launch_kernel(norm_rows_kernel<TO>, dim3(count), dim3(sn_threads(cols)), smem, st, stream, rows, w,
                            (TO*)out, cols, src_rows, eps, center, status, alpha, b);
}

extern "C" int ullm_norm_rows(int dtype, const float* stream, const int* rows, const float* w, void* out, int count,
                              int cols, int src_rows, float eps, int center, int* status, void* stream_handle,
                              const float* alpha, const float* b) {
  cudaStream_t st = (cudaStream_t)stream_handle;
  if (count < 0 || cols <= 0 || src_rows < 0 || center < 0 || center > 2) return ULLM_ERR_BAD_SIZE;
  if (center == 2 && (alpha == nullptr || b == nullptr)) return ULLM_ERR_BAD_SIZE;
  if (count == 0) return ULLM_OK;
  if (dtype == ULLM_DTYPE_F32)
    return norm_rows_launch<float>(stream, rows, w, out, count, cols, src_rows, eps, center, status, alpha, b, st);
  if (dtype == ULLM_DTYPE_BF16)
    return norm_rows_launch<__nv_bfloat16>(stream, rows, w, out, count, cols, src_rows, eps, center, status, alpha, b, st);
  if (dtype == ULLM_DTYPE_F16)
    return norm_rows_launch<__half>(stream, rows, w, out, count, cols, src_rows, eps, center, status, alpha, b, st);
  return ULLM_ERR_BAD_DTYPE;
}

template <typename T>
static int pair_norm_launch(const void* a, const void* b, const float* wa, const float* wb, int rows, int cols, float eps,
                            float mult, float* stream, void* rows_out, const float* w2, float eps2, int kind2,
                            const float* alpha2, const float* b2, void* out, const float* wo, float eps_o, float mult_o,
                            cudaStream_t st) {
  const size_t smem = 2 * (size_t)cols * sizeof(float);
  if (smem > SN_MAX_SMEM) return ULLM_ERR_UNSUPPORTED;
  constexpr int V = 16 / (int)sizeof(T);
  const bool wide = cols % V == 0 && (((uintptr_t)a | (uintptr_t)b | (uintptr_t)wa | (uintptr_t)wb | (uintptr_t)stream |
                                       (uintptr_t)rows_out | (uintptr_t)w2 | (uintptr_t)b2 | (uintptr_t)out |
                                       (uintptr_t)wo) & 15) == 0;
  int threads = 32;
  while (threads < 512 && threads * (wide ? V : 1) < cols) threads <<= 1;
#define PN_GO(VEC)                                                                                                    \
  {                                                                                                                   \
    const int rc = sn_allow_smem(pair_norm_add_norm_kernel<T, VEC>, smem);                                            \
    if (rc != ULLM_OK) return rc;                                                                                     \
    return ullm_launch_kernel(pair_norm_add_norm_kernel<T, VEC>, dim3(rows), dim3(threads), smem, st, (const T*)a,    \
                              (const T*)b, wa, wb, cols, eps, mult, stream, (T*)rows_out, w2, eps2, kind2, alpha2, b2, \
                              (T*)out, wo, eps_o, mult_o);                                                                               \
  }
  if (wide) PN_GO(V);
  PN_GO(1);
#undef PN_GO
}

// a, b [rows, cols] in the engine's dtype; `stream` (32-bit, updated in place) and `rows_out` (engine's dtype): at least
// one.  `out` with `w2` (null: none): the next norm of the updated rows; `kind2` 0: RMS, 1: centred, 2: tanh with `alpha2`
// (one number) and `b2`, 3: the rows as they are, rounded.  `wo` (null: none): the outer norm of the sum.
extern "C" int ullm_pair_norm_add_norm(int dtype, const void* a, const void* b, const float* wa, const float* wb, int rows,
                                       int cols, float eps, float mult, float* stream, void* rows_out, const float* w2,
                                       float eps2, int kind2, const float* alpha2, const float* b2, void* out,
                                       const float* wo, float eps_o, float mult_o, void* stream_handle) {
  cudaStream_t st = (cudaStream_t)stream_handle;
  if (rows < 0 || cols <= 0 || a == nullptr || b == nullptr || wa == nullptr || wb == nullptr ||
      (stream == nullptr && rows_out == nullptr) || (out != nullptr && w2 == nullptr && kind2 != 3) || kind2 < 0 || kind2 > 3 ||
      (out != nullptr && kind2 == 2 && (alpha2 == nullptr || b2 == nullptr)))
    return ULLM_ERR_BAD_SIZE;
  if (rows == 0) return ULLM_OK;
#define PN_ARGS a, b, wa, wb, rows, cols, eps, mult, stream, rows_out, w2, eps2, kind2, alpha2, b2, out, wo, eps_o, mult_o, st
  if (dtype == ULLM_DTYPE_F32) return pair_norm_launch<float>(PN_ARGS);
  if (dtype == ULLM_DTYPE_BF16) return pair_norm_launch<__nv_bfloat16>(PN_ARGS);
  if (dtype == ULLM_DTYPE_F16) return pair_norm_launch<__half>(PN_ARGS);
#undef PN_ARGS
  return ULLM_ERR_BAD_DTYPE;
}

// out = act(in) element by element; `pq`: the activation's two numbers (32-bit, on the device).
extern "C" int ullm_xielu(int dtype, const void* in, void* out, long long n, const float* pq, void* stream_handle) {
  cudaStream_t st = (cudaStream_t)stream_handle;
  if (n < 0 || pq == nullptr) return ULLM_ERR_BAD_SIZE;
  if (n == 0) return ULLM_OK;
  long long blocks = (n + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  const dim3 grid((int)blocks), block(256);
  if (dtype == ULLM_DTYPE_F32)
    return ullm_launch_kernel(xielu_kernel<float>, grid, block, 0, st, (const float*)in, (float*)out, n, pq);
  if (dtype == ULLM_DTYPE_BF16)
    return ullm_launch_kernel(xielu_kernel<__nv_bfloat16>, grid, block, 0, st, (const __nv_bfloat16*)in,
                              (__nv_bfloat16*)out, n, pq);
  if (dtype == ULLM_DTYPE_F16)
    return ullm_launch_kernel(xielu_kernel<__half>, grid, block, 0, st, (const __half*)in, (__half*)out, n, pq);
  return ULLM_ERR_BAD_DTYPE;
}

template <typename T>
static int relu2_launch(const void* in, void* out, long long n, cudaStream_t st) {
  constexpr int V = 16 / (int)sizeof(T);
  const bool wide = n % V == 0 && (((uintptr_t)in | (uintptr_t)out) & 15) == 0;
  long long blocks = (n / (wide ? V : 1) + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (wide) return ullm_launch_kernel(relu2_kernel<T, V>, dim3((int)blocks), dim3(256), 0, st, (const T*)in, (T*)out, n);
  return ullm_launch_kernel(relu2_kernel<T, 1>, dim3((int)blocks), dim3(256), 0, st, (const T*)in, (T*)out, n);
}

// out = max(in, 0)^2 element by element (`out` may be `in`).
extern "C" int ullm_relu2(int dtype, const void* in, void* out, long long n, void* stream_handle) {
  cudaStream_t st = (cudaStream_t)stream_handle;
  if (n < 0) return ULLM_ERR_BAD_SIZE;
  if (n == 0) return ULLM_OK;
  if (dtype == ULLM_DTYPE_F32) return relu2_launch<float>(in, out, n, st);
  if (dtype == ULLM_DTYPE_BF16) return relu2_launch<__nv_bfloat16>(in, out, n, st);
  if (dtype == ULLM_DTYPE_F16) return relu2_launch<__half>(in, out, n, st);
  return ULLM_ERR_BAD_DTYPE;
}

template <typename T, int ACT>
static int act_rows_launch(const void* in, long long in_stride, void* out, long long out_stride, int rows, int cols,
                           cudaStream_t st) {
  constexpr int V = 16 / (int)sizeof(T);
  const bool wide = cols % V == 0 && in_stride % V == 0 && out_stride % V == 0 && (((uintptr_t)in | (uintptr_t)out) & 15) == 0;
  const int per_row = wide ? cols / V : cols;
  const long long pieces = (long long)rows * per_row;
  long long blocks = (pieces + 127) / 128;
  if (blocks > 148 * 32) blocks = 148 * 32;
  if (wide)
    return ullm_launch_kernel(act_rows_kernel<T, V, ACT>, dim3((int)blocks), dim3(128), 0, st, (const T*)in, in_stride,
                              (T*)out, out_stride, pieces, per_row);
  return ullm_launch_kernel(act_rows_kernel<T, 1, ACT>, dim3((int)blocks), dim3(128), 0, st, (const T*)in, in_stride,
                            (T*)out, out_stride, pieces, per_row);
}

// `act` 0: silu, 1: the exact gelu; rows of `cols` elements, strides in elements, `out` may be `in`.
extern "C" int ullm_act_rows(int dtype, int act, const void* in, long long in_stride, void* out, long long out_stride,
                             int rows, int cols, void* stream_handle) {
  cudaStream_t st = (cudaStream_t)stream_handle;
  if (rows < 0 || cols <= 0 || in_stride < cols || out_stride < cols || act < 0 || act > 1) return ULLM_ERR_BAD_SIZE;
  if (rows == 0) return ULLM_OK;
#define AR_GO(T)                                                                                         \
  return act == 0 ? act_rows_launch<T, 0>(in, in_stride, out, out_stride, rows, cols, st)                \
                  : act_rows_launch<T, 1>(in, in_stride, out, out_stride, rows, cols, st)
  if (dtype == ULLM_DTYPE_F32) AR_GO(float);
  if (dtype == ULLM_DTYPE_BF16) AR_GO(__nv_bfloat16);
  if (dtype == ULLM_DTYPE_F16) AR_GO(__half);
#undef AR_GO
  return ULLM_ERR_BAD_DTYPE;
}
