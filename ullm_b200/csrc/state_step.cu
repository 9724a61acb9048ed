// One token of every request through a matrix state per head, for decode steps: the recurrences of csrc/ssd.cu and
// csrc/gla.cu where every request of the step brings exactly one token.
//
//   S' = diag(a) S + k v^T,   y = S'^T q          or, with a bonus u:   y = (S + diag(u) k v^T)^T q
//
//   SSD   a = exp(log_decay) (one number per head), k = dt B, v = x, q = C (of the head's group), y += D x; optionally a
//         silu on x, B and C as they are read
//   GLA   a per key channel: a 32-bit row of decays, or exp(logsigmoid(z + bias) / tau) of it; q = q_scale * (projected query)
//
// A step reads and writes the whole state once and does little else, so the kernel is built around that stream: the state
// row S^T is [columns][n], `lanes` neighbouring lanes (a power of two, four entries of n each, 16-byte accesses) own a
// column, a warp holds 32 / lanes columns at a time and has SST_U such sets in flight; decays, keys and queries wait in
// registers.  Sums over n are shuffles.  One block per (request, head, tile of columns).
#include "common.cuh"

#define SST_WARPS 4
#define SST_U 8

struct StepArgs {
  const void* rows;  // [requests][row_stride]: what v, k and q are read from
  long long row_stride;
  int v_off, k_off, q_off;
  int heads, n, cols, per_group;  // heads of a group share k and q
  const float* decay;             // SSD: log_decay [.][heads]; GLA: decays (or z) [.][heads * n]
  long long decay_stride;
  const float* dt;                // SSD: steps, rows as `decay`
  const float* skip;              // SSD: D [heads]
  int silu_in;
  const float* z_bias;            // GLA, inv_tau > 0
  float inv_tau, q_scale;
  const float* bonus;             // GLA: [heads * n] or null
  float* state;
  long long state_stride;
  const int* req_slots;
  const int* token_req;
  float* out;                     // [requests][heads * cols]
  int num_slots;
  int* status;
};

// NI: pieces of 4 * lanes entries of n that a lane walks (n <= 4 * lanes * NI)
template <typename T, bool GLA, int NI>
__global__ void __launch_bounds__(SST_WARPS * 32) state_step_kernel(const StepArgs p, int lanes, int col_tile) {
  pdl_launch_dependents();
  pdl_wait();
  const int req = blockIdx.z, head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int sub = lane / lanes, ln = lane - sub * lanes, per_pass = 32 / lanes;
  const int col_end = min(p.cols, (int)(blockIdx.x + 1) * col_tile);
  float* out = p.out + ((long long)req * p.heads + head) * p.cols;
  if (p.token_req[req] < 0) {  // a row that belongs to no request: zeros out, no state touched
    for (int c = blockIdx.x * col_tile + threadIdx.x; c < col_end; c += blockDim.x) out[c] = 0.f;
    return;
  }
  const int slot = p.req_slots[req];
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0) ullm_report(p.status, ULLM_STATUS_SLOT, req, slot);
    return;
  }
  const T* row = (const T*)p.rows + (long long)req * p.row_stride;
  const int kh = head / p.per_group;
  float a[NI][4], k[NI][4], q[NI][4], u[NI][4];
  float skip = 0.f;
  if (!GLA) skip = p.skip[head];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int e0 = (i * lanes + ln) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) a[i][e] = k[i][e] = q[i][e] = u[i][e] = 0.f;
    if (e0 >= p.n) continue;
    if (GLA) {
      const float4 w = *reinterpret_cast<const float4*>(p.decay + req * p.decay_stride + head * p.n + e0);
      a[i][0] = w.x, a[i][1] = w.y, a[i][2] = w.z, a[i][3] = w.w;
      if (p.inv_tau > 0.f) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float z = a[i][e] + (p.z_bias != nullptr ? p.z_bias[head * p.n + e0 + e] : 0.f);
          a[i][e] = expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * p.inv_tau);
        }
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      k[i][e] = to_f32(row[p.k_off + kh * p.n + e0 + e]);
      q[i][e] = to_f32(row[p.q_off + kh * p.n + e0 + e]);
      if (GLA) {
        q[i][e] *= p.q_scale;
        if (p.bonus != nullptr) u[i][e] = p.bonus[head * p.n + e0 + e];
      } else if (p.silu_in) {
        k[i][e] = act_silu(k[i][e]);
        q[i][e] = act_silu(q[i][e]);
      }
    }
  }
  if (!GLA) {
    const float w = expf(p.decay[req * p.decay_stride + head]), d = p.dt[req * p.decay_stride + head];
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        a[i][e] = w;
        k[i][e] *= d;
      }
  }
  float* st = p.state + (long long)slot * p.state_stride + (long long)head * p.cols * p.n;
  const bool has_bonus = GLA && p.bonus != nullptr;
  // the warp's columns: sets of per_pass, SST_U sets at a time
  for (int c0 = blockIdx.x * col_tile + warp * per_pass; c0 < col_end; c0 += SST_WARPS * per_pass * SST_U) {
    float4 s[SST_U][NI];
    float v[SST_U], y[SST_U];
#pragma unroll
    for (int j = 0; j < SST_U; ++j) {
      const int c = c0 + j * SST_WARPS * per_pass + sub;
      v[j] = 0.f;
      if (c < col_end) {
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          const int e0 = (i * lanes + ln) * 4;
          s[j][i] = e0 < p.n ? *reinterpret_cast<const float4*>(st + (long long)c * p.n + e0) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        v[j] = to_f32(row[p.v_off + head * p.cols + c]);
        if (!GLA && p.silu_in) v[j] = act_silu(v[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < SST_U; ++j) {
      const int c = c0 + j * SST_WARPS * per_pass + sub;
      y[j] = 0.f;
      if (c < col_end) {
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          float x[4] = {s[j][i].x, s[j][i].y, s[j][i].z, s[j][i].w};
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float kv = k[i][e] * v[j];
            if (has_bonus) y[j] = fmaf(fmaf(u[i][e], kv, x[e]), q[i][e], y[j]);
            x[e] = fmaf(a[i][e], x[e], kv);
            if (!has_bonus) y[j] = fmaf(x[e], q[i][e], y[j]);
          }
          const int e0 = (i * lanes + ln) * 4;
          if (e0 < p.n) *reinterpret_cast<float4*>(st + (long long)c * p.n + e0) = make_float4(x[0], x[1], x[2], x[3]);
        }
      }
    }
    for (int o = lanes >> 1; o > 0; o >>= 1) {
#pragma unroll
      for (int j = 0; j < SST_U; ++j) y[j] += __shfl_xor_sync(0xffffffffu, y[j], o);
    }
    if (ln == 0) {
#pragma unroll
      for (int j = 0; j < SST_U; ++j) {
        const int c = c0 + j * SST_WARPS * per_pass + sub;
        if (c < col_end) out[c] = GLA ? y[j] : fmaf(skip, v[j], y[j]);
      }
    }
  }
}

template <typename T, bool GLA>
static int step_go(const StepArgs& p, int requests, cudaStream_t st) {
  int lanes = 1;
  while (lanes < 32 && lanes * 4 < p.n) lanes <<= 1;
  const int ni = (p.n + lanes * 4 - 1) / (lanes * 4);
  // columns per block: as many as one turn of its warps takes, fewer where the blocks would not fill the SMs twice
  int sms = 148, dev = 0;
  if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  const int set = SST_WARPS * (32 / lanes);
  int tile = set * SST_U;
  while (tile > set && (long long)((p.cols + tile - 1) / tile) * p.heads * requests < 4LL * sms) tile >>= 1;
  const dim3 grid((p.cols + tile - 1) / tile, p.heads, requests), block(SST_WARPS * 32);
#define SST_GO(NI) return ullm_launch_kernel(state_step_kernel<T, GLA, NI>, grid, block, 0, st, p, lanes, tile)
  if (ni == 1) SST_GO(1);
  if (ni == 2) SST_GO(2);
  if (ni <= 4) SST_GO(4);
#undef SST_GO
  return ULLM_ERR_UNSUPPORTED;
}

static bool step_sizes_ok(int requests, int heads, int n, int cols, const float* state, long long state_stride) {
  return requests > 0 && requests <= 65535 && heads > 0 && heads <= 65535 && n > 0 && n % 4 == 0 && n <= 512 && cols > 0 &&
         state_stride % 4 == 0 && state_stride >= (long long)heads * n * cols && ((uintptr_t)state & 15) == 0;
}

// `ullm_ssd_recurrence` for steps in which every request has one token.  ULLM_ERR_UNSUPPORTED (nothing has run): sizes or
// alignments that the token-by-token kernel takes.
extern "C" int ullm_ssd_step(int dtype, const void* xbc, long long row_stride, int b_off, int c_off, const float* dt,
                             const float* log_decay, const float* d_skip, float* state, long long state_stride,
                             const int* req_slots, const int* token_req, float* out, int requests, int heads, int n_state,
                             int pdim, int groups, int num_slots, int* status, void* stream, long long dt_stride,
                             int silu_in) {
  if (groups <= 0 || heads % groups || !step_sizes_ok(requests, heads, n_state, pdim, state, state_stride)) return ULLM_ERR_UNSUPPORTED;
  StepArgs p = {};
  p.rows = xbc;
  p.row_stride = row_stride;
  p.v_off = 0;
  p.k_off = b_off;
  p.q_off = c_off;
  p.heads = heads;
  p.n = n_state;
  p.cols = pdim;
  p.per_group = heads / groups;
  p.decay = log_decay;
  p.decay_stride = dt_stride;
  p.dt = dt;
  p.skip = d_skip;
  p.silu_in = silu_in;
  p.state = state;
  p.state_stride = state_stride;
  p.req_slots = req_slots;
  p.token_req = token_req;
  p.out = out;
  p.num_slots = num_slots;
  p.status = status;
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == ULLM_DTYPE_F32) return step_go<float, false>(p, requests, st);
  if (dtype == ULLM_DTYPE_BF16) return step_go<__nv_bfloat16, false>(p, requests, st);
  if (dtype == ULLM_DTYPE_F16) return step_go<__half, false>(p, requests, st);
  return ULLM_ERR_BAD_DTYPE;
}

// `ullm_gla_recurrence` for such steps; `z` is left as it is.
extern "C" int ullm_gla_step(int dtype, const void* qkv, long long row_stride, int q_off, int k_off, int v_off, const float* z,
                             long long z_stride, const float* z_bias, float inv_tau, float q_scale, float* state,
                             long long state_stride, const int* req_slots, const int* token_req, float* out, int requests,
                             int heads, int dim, int vdim, int num_slots, int* status, void* stream, const float* bonus) {
  if (!step_sizes_ok(requests, heads, dim, vdim, state, state_stride) || z_stride % 4 || ((uintptr_t)z & 15)) return ULLM_ERR_UNSUPPORTED;
  StepArgs p = {};
  p.rows = qkv;
  p.row_stride = row_stride;
  p.v_off = v_off;
  p.k_off = k_off;
  p.q_off = q_off;
  p.heads = heads;
  p.n = dim;
  p.cols = vdim;
  p.per_group = 1;
  p.decay = z;
  p.decay_stride = z_stride;
  p.z_bias = z_bias;
  p.inv_tau = inv_tau;
  p.q_scale = q_scale;
  p.bonus = bonus;
  p.state = state;
  p.state_stride = state_stride;
  p.req_slots = req_slots;
  p.token_req = token_req;
  p.out = out;
  p.num_slots = num_slots;
  p.status = status;
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == ULLM_DTYPE_F32) return step_go<float, true>(p, requests, st);
  if (dtype == ULLM_DTYPE_BF16) return step_go<__nv_bfloat16, true>(p, requests, st);
  if (dtype == ULLM_DTYPE_F16) return step_go<__half, true>(p, requests, st);
  return ULLM_ERR_BAD_DTYPE;
}
