// The recurrence of csrc/gla.cu (a decay per key channel, with or without the bonus of the current token) for prompt
// portions in bfloat16, GCH_Q tokens at a time on the tensor cores, all chunks side by side.
//
// With w_t the decays, W(a, b) = prod_{a < q <= b} w_q (a product per key channel) and S the state in front of the chunk
// (first token 1):
//
//   without bonus   y_t = (q_t W(0, t))^T S + sum_{s <= t} (q_t . (W(s, t) k_s)) v_s
//   with bonus u    y_t = (q_t W(0, t-1))^T S + sum_{s < t} (q_t . (W(s, t-1) k_s)) v_s + (q_t . (u k_t)) v_t
//   S'              = W(0, Q) S + sum_s (W(s, Q) k_s) v_s^T
//
// Three kernels: `gla_fold` forms every chunk's own contribution to the state and its total decay, `gla_scan` walks the chunks
// of a request element by element and leaves in front of every chunk the state it starts from, `gla_out` forms the outputs.
//
// Decays enter as products only, never as quotients or differences of logarithms, so nothing overflows and nothing cancels
// however strong they are: a chunk is cut into stretches of GCH_SUB tokens; a query meets the keys of an EARLIER stretch as
// (q_t W(start of its stretch, t)) . (decays of the stretches between) . (W(s, end of the key's stretch) k_s), a matrix
// product; the keys of its own stretch one by one in 32-bit, the product of decays carried from token to token.
//
// Precision: v is an exact bfloat16 operand; every 32-bit operand (weighted queries and keys, scores, the state) enters as
// TWO bfloat16 terms, rounded value and rounded rest; accumulators, decays and states are 32-bit.
//
// mma.sync m16n8k16; a block of four warps owns (chunk, head), warp w the chunk's rows 16 w .. 16 w + 15.
#include "common.cuh"

#define GCH_Q 64
#define GCH_SUB 8
#define GCH_SUBS (GCH_Q / GCH_SUB)
#define GCH_THREADS 128
#define GCH_MAX_DIM 256

__device__ __forceinline__ void gch_ldsm4t(unsigned (&r)[4], const void* p) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(s));
}
__device__ __forceinline__ void gch_mma(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void gch_split(float v0, float v1, unsigned& hi, unsigned& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(v0, v1);
  const __nv_bfloat162 l = __floats2bfloat162_rn(v0 - __bfloat162float(h.x), v1 - __bfloat162float(h.y));
  hi = *reinterpret_cast<const unsigned*>(&h);
  lo = *reinterpret_cast<const unsigned*>(&l);
}

// Chunk `tile` of the step: its first token and its tokens (0: there is no such chunk).  Chunks are counted over the
// requests that bring more than `least` tokens, from each request's first token of the step.
__device__ __forceinline__ int gch_find(int tile, const int* cu_q, int requests, int least, int& t0) {
  for (int i = 0; i < requests; ++i) {
    const int b = cu_q[i], n = cu_q[i + 1] - b;
    if (n <= least) continue;
    const int nt = (n + GCH_Q - 1) / GCH_Q;
    if (tile < nt) {
      t0 = b + tile * GCH_Q;
      return min(GCH_Q, n - tile * GCH_Q);
    }
    tile -= nt;
  }
  return 0;
}

// v of the chunk, [GCH_Q][vdim + 8] bfloat16, rows past the chunk's end zero
__device__ __forceinline__ void gch_load_v(__nv_bfloat16* v_s, const __nv_bfloat16* v, long long row_stride, int vdim, int cn) {
  const int pieces = vdim >> 3;
  for (int i = threadIdx.x; i < GCH_Q * pieces; i += GCH_THREADS) {
    const int row = i / pieces, ch = (i - row * pieces) << 3;
    uint4 x = make_uint4(0, 0, 0, 0);
    if (row < cn) x = *reinterpret_cast<const uint4*>(v + (long long)row * row_stride + ch);
    *reinterpret_cast<uint4*>(v_s + row * (vdim + 8) + ch) = x;
  }
}

// fold[(tile * heads + head)][vdim][dim] = sum_s v_s (W(s, Q) k_s)^T;  total[(tile * heads + head)][dim] = W(0, Q)
__global__ void __launch_bounds__(GCH_THREADS)
gla_fold_kernel(const __nv_bfloat16* __restrict__ qkv, long long row_stride, int k_off, int v_off,
                const float* __restrict__ decay, long long decay_stride, const int* __restrict__ cu_q,
                const int* __restrict__ token_req, int requests, int least, int heads, int dim, int vdim,
                float* __restrict__ fold, float* __restrict__ total) {
  extern __shared__ __align__(16) unsigned char gch_smem[];
  pdl_launch_dependents();
  pdl_wait();
  int t0 = 0;
  const int tile = blockIdx.x, head = blockIdx.y;
  const int cn = gch_find(tile, cu_q, requests, least, t0);
  if (cn == 0 || token_req[t0] < 0) return;
  const int ks = dim + 4;  // (two rows are 8 banks apart: a fragment's reads do not meet)
  float* kq = reinterpret_cast<float*>(gch_smem);                             // [GCH_Q][ks]: W(s, end of its stretch) k_s
  float* tot = kq + GCH_Q * ks;                                               // [GCH_SUBS][dim]
  __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(tot + GCH_SUBS * dim);  // [GCH_Q][vdim + 8]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  gch_load_v(v_s, qkv + (long long)t0 * row_stride + v_off + head * vdim, row_stride, vdim, cn);
  for (int i = tid; i < GCH_SUBS * dim; i += GCH_THREADS) {
    const int sub = i / dim, ch = i - sub * dim, r0 = sub * GCH_SUB;
    float w[GCH_SUB], k[GCH_SUB];
#pragma unroll
    for (int j = 0; j < GCH_SUB; ++j) {
      const long long t = t0 + r0 + j;
      const bool ok = r0 + j < cn;
      w[j] = ok ? decay[t * decay_stride + head * dim + ch] : 1.f;
      k[j] = ok ? __bfloat162float(qkv[t * row_stride + k_off + head * dim + ch]) : 0.f;
    }
    float q = 1.f;
#pragma unroll
    for (int j = GCH_SUB - 1; j >= 0; --j) {
      kq[(r0 + j) * ks + ch] = k[j] * q;
      q *= w[j];
    }
    tot[sub * dim + ch] = q;
  }
  __syncthreads();
  // what follows a stretch inside the chunk: suffix products of the totals; the whole product is the chunk's total
  for (int ch = tid; ch < dim; ch += GCH_THREADS) {
    float f = 1.f;
#pragma unroll
    for (int sub = GCH_SUBS - 1; sub >= 0; --sub) {
      const float x = tot[sub * dim + ch];
      tot[sub * dim + ch] = f;
      f *= x;
    }
    total[((long long)tile * heads + head) * dim + ch] = f;
  }
  __syncthreads();
  float* out = fold + ((long long)tile * heads + head) * vdim * dim;
  const int mat = lane >> 3;
  for (int n0 = warp * 8; n0 < dim; n0 += 32) {  // eight key channels of the state
    const int ch = n0 + (lane >> 2);
    unsigned bh[4][2], bl[4][2];
#pragma unroll
    for (int s = 0; s < 4; ++s)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int r = s * 16 + h * 8 + (lane & 3) * 2;
        const float f = tot[(s * 2 + h) * dim + ch];
        gch_split(kq[r * ks + ch] * f, kq[(r + 1) * ks + ch] * f, bh[s][h], bl[s][h]);
      }
    for (int m0 = 0; m0 < vdim; m0 += 16) {
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int s = 0; s < 4; ++s) {
        unsigned a[4];
        gch_ldsm4t(a, v_s + (s * 16 + (mat >> 1) * 8 + (lane & 7)) * (vdim + 8) + m0 + (mat & 1) * 8);
        gch_mma(acc, a, bh[s][0], bh[s][1]);
        gch_mma(acc, a, bl[s][0], bl[s][1]);
      }
#pragma unroll
      for (int h = 0; h < 2; ++h)
        *reinterpret_cast<float2*>(out + (long long)(m0 + (lane >> 2) + 8 * h) * dim + n0 + (lane & 3) * 2) =
            make_float2(acc[2 * h], acc[2 * h + 1]);
    }
  }
}

// fold <- the state in front of every chunk, as pairs of key channels: (two rounded values, two rounded rests), the operands
// that `gla_out` needs; state <- the state behind the last.  Two neighbouring key channels per thread.
__global__ void gla_scan_kernel(float* __restrict__ fold, const float* __restrict__ total, float* __restrict__ state,
                                long long state_stride, const int* __restrict__ cu_q, const int* __restrict__ req_slots,
                                const int* __restrict__ token_req, int least, int heads, int dim, int vdim,
                                int num_slots, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int req = blockIdx.z, head = blockIdx.y;
  const int t0 = cu_q[req], n = cu_q[req + 1] - t0;
  if (n <= least || token_req[t0] < 0) return;
  const int slot = req_slots[req];
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0) ullm_report(status, ULLM_STATUS_SLOT, req, slot);
    return;
  }
  int tile = 0;
  for (int i = 0; i < req; ++i) {
    const int m = cu_q[i + 1] - cu_q[i];
    if (m > least) tile += (m + GCH_Q - 1) / GCH_Q;
  }
  const int e = (blockIdx.x * blockDim.x + threadIdx.x) * 2;
  if (e >= dim * vdim) return;
  const int chunks = (n + GCH_Q - 1) / GCH_Q;
  const long long step = (long long)heads * dim * vdim;
  float* f = fold + ((long long)tile * heads + head) * dim * vdim + e;
  const float* w = total + ((long long)tile * heads + head) * dim + e % dim;
  float2* st = reinterpret_cast<float2*>(state + (long long)slot * state_stride + (long long)head * dim * vdim + e);
  float2 s = *st;
  constexpr int U = 8;
  for (int c0 = 0; c0 < chunks; c0 += U) {
    float2 d[U], a[U];
#pragma unroll
    for (int j = 0; j < U; ++j)
      if (c0 + j < chunks) {
        d[j] = *reinterpret_cast<const float2*>(f + (c0 + j) * step);
        a[j] = *reinterpret_cast<const float2*>(w + (long long)(c0 + j) * heads * dim);
      }
#pragma unroll
    for (int j = 0; j < U; ++j)
      if (c0 + j < chunks) {
        uint2 terms;
        gch_split(s.x, s.y, terms.x, terms.y);
        *reinterpret_cast<uint2*>(f + (c0 + j) * step) = terms;
        s.x = fmaf(a[j].x, s.x, d[j].x);
        s.y = fmaf(a[j].y, s.y, d[j].y);
      }
  }
  *st = s;
}

// A warp's 16 rows are two stretches, i0 and i0 + 1; its queries are weighted from the start of stretch i0 on.
template <bool BONUS>
__global__ void __launch_bounds__(GCH_THREADS, 3)
gla_out_kernel(const __nv_bfloat16* __restrict__ qkv, long long row_stride, int q_off, int k_off, int v_off,
               const float* __restrict__ decay, long long decay_stride, const float* __restrict__ bonus, float q_scale,
               const int* __restrict__ cu_q, const int* __restrict__ token_req, int requests, int least, int heads, int dim,
               int vdim, const float* __restrict__ fold, float* __restrict__ out) {
  extern __shared__ __align__(16) unsigned char gch_smem[];
  pdl_launch_dependents();
  pdl_wait();
  int t0 = 0;
  const int tile = blockIdx.x, head = blockIdx.y;
  const int cn = gch_find(tile, cu_q, requests, least, t0);
  if (cn == 0 || token_req[t0] < 0) return;
  const int ks = dim + 4, kb = dim + 8;
  float* rp = reinterpret_cast<float*>(gch_smem);                     // [GCH_Q][ks]: q, then weighted q
  float* kq = rp + GCH_Q * ks;                                        // [GCH_Q][ks]: decays, then weighted k
  float* tot = kq + GCH_Q * ks;                                       // [GCH_SUBS][dim]
  float* diag = tot + GCH_SUBS * dim;                                 // [GCH_SUBS][8][10]: scores inside the stretches
  __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(diag + GCH_SUBS * 80);  // [GCH_Q][vdim + 8]
  __nv_bfloat16* k_s = v_s + GCH_Q * (vdim + 8);                      // [GCH_Q][kb]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  gch_load_v(v_s, qkv + (long long)t0 * row_stride + v_off + head * vdim, row_stride, vdim, cn);
  {
    const int pieces = dim >> 3;
    for (int i = tid; i < GCH_Q * pieces; i += GCH_THREADS) {
      const int row = i / pieces, ch = (i - row * pieces) << 3;
      float q[8];
      float4 w0 = make_float4(1.f, 1.f, 1.f, 1.f), w1 = w0;
      uint4 k = make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int j = 0; j < 8; ++j) q[j] = 0.f;
      if (row < cn) {
        const __nv_bfloat16* src = qkv + (long long)(t0 + row) * row_stride + head * dim + ch;
        load_vec<__nv_bfloat16, 8>(src + q_off, q);
        k = *reinterpret_cast<const uint4*>(src + k_off);
        const float4* wp = reinterpret_cast<const float4*>(decay + (long long)(t0 + row) * decay_stride + head * dim + ch);
        w0 = wp[0];
        w1 = wp[1];
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) q[j] *= q_scale;
      store_vec32<8>(rp + row * ks + ch, q);
      *reinterpret_cast<float4*>(kq + row * ks + ch) = w0;
      *reinterpret_cast<float4*>(kq + row * ks + ch + 4) = w1;
      *reinterpret_cast<uint4*>(k_s + row * kb + ch) = k;
    }
  }
  __syncthreads();
  // ---- scores inside the warp's two stretches: a lane owns key s of one of them and every second pair of channels ----
  {
    const int s = lane & 7, blk = (lane >> 3) & 1, half = lane >> 4, r0 = warp * 16 + blk * 8;
    float sc[GCH_SUB], own = 0.f;
#pragma unroll
    for (int t = 0; t < GCH_SUB; ++t) sc[t] = 0.f;
    const int quads = dim >> 2;
    int c = blk;  // (the two stretches' rows lie on the same banks: they take the channels in turn)
    for (int i = 0; i < quads; ++i) {
      const int ch = 4 * c + 2 * half;
      if (++c == quads) c = 0;
      const __nv_bfloat162 kv = *reinterpret_cast<const __nv_bfloat162*>(k_s + (r0 + s) * kb + ch);
      const float2 qs = *reinterpret_cast<const float2*>(rp + (r0 + s) * ks + ch);
      float ex = __bfloat162float(kv.x), ey = __bfloat162float(kv.y);
      float2 u = make_float2(1.f, 1.f);
      if (BONUS) u = *reinterpret_cast<const float2*>(bonus + head * dim + ch);
      own = fmaf(qs.x * u.x, ex, own);
      own = fmaf(qs.y * u.y, ey, own);
      const float* qp = rp + r0 * ks + ch;
      const float* wp = kq + r0 * ks + ch;
#pragma unroll
      for (int t = 1; t < GCH_SUB; ++t) {  // (what is formed for t <= s is thrown away below)
        const float2 q = *reinterpret_cast<const float2*>(qp + t * ks), w = *reinterpret_cast<const float2*>(wp + t * ks);
        if (!BONUS && t > s) {
          ex *= w.x;
          ey *= w.y;
        }
        sc[t] = fmaf(q.x, ex, sc[t]);
        sc[t] = fmaf(q.y, ey, sc[t]);
        if (BONUS && t > s) {
          ex *= w.x;
          ey *= w.y;
        }
      }
    }
    own += __shfl_xor_sync(0xffffffffu, own, 16);
#pragma unroll
    for (int t = 0; t < GCH_SUB; ++t) {
      sc[t] += __shfl_xor_sync(0xffffffffu, sc[t], 16);
      if (half == 0) diag[(warp * 2 + blk) * 80 + t * 10 + s] = t > s ? sc[t] : (t == s ? own : 0.f);
    }
  }
  __syncthreads();
  // ---- q <- W(start of its stretch, t or t - 1) q,  decays <- (rounded, rest) of W(s, end of its stretch) k ----------
  for (int i = tid; i < GCH_SUBS * (dim >> 1); i += GCH_THREADS) {
    const int sub = i / (dim >> 1), ch = (i - sub * (dim >> 1)) * 2, r0 = sub * GCH_SUB;
    float2 w[GCH_SUB];
    float2 p = make_float2(1.f, 1.f);
#pragma unroll
    for (int j = 0; j < GCH_SUB; ++j) {
      w[j] = *reinterpret_cast<const float2*>(kq + (r0 + j) * ks + ch);
      float2* qp = reinterpret_cast<float2*>(rp + (r0 + j) * ks + ch);
      float2 q = *qp;
      if (!BONUS) p.x *= w[j].x, p.y *= w[j].y;
      q.x *= p.x;
      q.y *= p.y;
      *qp = q;
      if (BONUS) p.x *= w[j].x, p.y *= w[j].y;
    }
    p = make_float2(1.f, 1.f);
#pragma unroll
    for (int j = GCH_SUB - 1; j >= 0; --j) {
      const __nv_bfloat162 kv = *reinterpret_cast<const __nv_bfloat162*>(k_s + (r0 + j) * kb + ch);
      *reinterpret_cast<float2*>(kq + (r0 + j) * ks + ch) = make_float2(__bfloat162float(kv.x) * p.x, __bfloat162float(kv.y) * p.y);
      p.x *= w[j].x, p.y *= w[j].y;
    }
    *reinterpret_cast<float2*>(tot + sub * dim + ch) = p;
  }
  __syncthreads();
  if (warp * 16 >= cn) return;
  const int i0 = 2 * warp, g = lane >> 2, cp = (lane & 3) * 2;
  // ---- scores against the stretches in front: acc[j] are the warp's 16 rows against stretch j ----------------------
  float acc[GCH_SUBS][4];
#pragma unroll
  for (int j = 0; j < GCH_SUBS; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  float near[4] = {0.f, 0.f, 0.f, 0.f};  // rows of stretch i0 + 1 against stretch i0
  for (int kk = 0; kk < dim; kk += 16) {
    float* r_lo = rp + (warp * 16 + g) * ks + kk + cp;  // rows of stretch i0
    float* r_hi = r_lo + 8 * ks;                        // rows of stretch i0 + 1
    float2 q0 = *reinterpret_cast<const float2*>(r_lo), q1 = *reinterpret_cast<const float2*>(r_hi),
           q2 = *reinterpret_cast<const float2*>(r_lo + 8), q3 = *reinterpret_cast<const float2*>(r_hi + 8);
    unsigned ah[4], al[4], bh[2], bl[2];
    {
      ah[0] = ah[2] = al[0] = al[2] = 0u;
      gch_split(q1.x, q1.y, ah[1], al[1]);
      gch_split(q3.x, q3.y, ah[3], al[3]);
      const float2 k0 = *reinterpret_cast<const float2*>(kq + (i0 * 8 + g) * ks + kk + cp);
      const float2 k1 = *reinterpret_cast<const float2*>(kq + (i0 * 8 + g) * ks + kk + cp + 8);
      gch_split(k0.x, k0.y, bh[0], bl[0]);
      gch_split(k1.x, k1.y, bh[1], bl[1]);
      gch_mma(near, ah, bh[0], bh[1]);
      gch_mma(near, ah, bl[0], bl[1]);
      gch_mma(near, al, bh[0], bh[1]);
    }
    const float2 d0 = *reinterpret_cast<const float2*>(tot + i0 * dim + kk + cp);
    const float2 d1 = *reinterpret_cast<const float2*>(tot + i0 * dim + kk + cp + 8);
    q1.x *= d0.x, q1.y *= d0.y;
    q3.x *= d1.x, q3.y *= d1.y;
    gch_split(q0.x, q0.y, ah[0], al[0]);
    gch_split(q1.x, q1.y, ah[1], al[1]);
    gch_split(q2.x, q2.y, ah[2], al[2]);
    gch_split(q3.x, q3.y, ah[3], al[3]);
    float2 f0 = make_float2(1.f, 1.f), f1 = f0;  // the decays between stretch j's end and stretch i0's start
#pragma unroll
    for (int jj = 0; jj < GCH_SUBS - 2; ++jj) {
      const int j = GCH_SUBS - 3 - jj;
      if (j < i0) {
        const float2 k0 = *reinterpret_cast<const float2*>(kq + (j * 8 + g) * ks + kk + cp);
        const float2 k1 = *reinterpret_cast<const float2*>(kq + (j * 8 + g) * ks + kk + cp + 8);
        gch_split(k0.x * f0.x, k0.y * f0.y, bh[0], bl[0]);
        gch_split(k1.x * f1.x, k1.y * f1.y, bh[1], bl[1]);
        gch_mma(acc[j], ah, bh[0], bh[1]);
        gch_mma(acc[j], ah, bl[0], bl[1]);
        gch_mma(acc[j], al, bh[0], bh[1]);
        const float2 e0 = *reinterpret_cast<const float2*>(tot + j * dim + kk + cp);
        const float2 e1 = *reinterpret_cast<const float2*>(tot + j * dim + kk + cp + 8);
        f0.x *= e0.x, f0.y *= e0.y;
        f1.x *= e1.x, f1.y *= e1.y;
      }
    }
    // weighted down to the chunk's start: what meets the state
    *reinterpret_cast<float2*>(r_lo) = make_float2(q0.x * f0.x, q0.y * f0.y);
    *reinterpret_cast<float2*>(r_hi) = make_float2(q1.x * f0.x, q1.y * f0.y);
    *reinterpret_cast<float2*>(r_lo + 8) = make_float2(q2.x * f1.x, q2.y * f1.y);
    *reinterpret_cast<float2*>(r_hi + 8) = make_float2(q3.x * f1.x, q3.y * f1.y);
  }
  {
    const float2 d0 = *reinterpret_cast<const float2*>(diag + i0 * 80 + g * 10 + cp);
    const float2 d1 = *reinterpret_cast<const float2*>(diag + (i0 + 1) * 80 + g * 10 + cp);
#pragma unroll
    for (int j = 0; j < GCH_SUBS; ++j) {  // (these places are still zero; sums, so that acc stays in registers)
      const float a = j == i0 ? 1.f : 0.f, b = j == i0 + 1 ? 1.f : 0.f;
      acc[j][0] = fmaf(a, d0.x, acc[j][0]);
      acc[j][1] = fmaf(a, d0.y, acc[j][1]);
      acc[j][2] = fmaf(a, near[2], fmaf(b, d1.x, acc[j][2]));
      acc[j][3] = fmaf(a, near[3], fmaf(b, d1.y, acc[j][3]));
    }
  }
  __syncwarp();
  // ---- outputs, 64 value columns at a time --------------------------------------------------------------------------
  const float* st = fold + ((long long)tile * heads + head) * vdim * dim;
  const int mat = lane >> 3;
  for (int n0 = 0; n0 < vdim; n0 += 64) {
    const int nt = min(8, (vdim - n0) >> 3);
    float y[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) y[n][0] = y[n][1] = y[n][2] = y[n][3] = 0.f;
#pragma unroll
    for (int s = 0; s < 4; ++s) {
      if (s <= warp) {
        unsigned ah[4], al[4];
        gch_split(acc[2 * s][0], acc[2 * s][1], ah[0], al[0]);
        gch_split(acc[2 * s][2], acc[2 * s][3], ah[1], al[1]);
        gch_split(acc[2 * s + 1][0], acc[2 * s + 1][1], ah[2], al[2]);
        gch_split(acc[2 * s + 1][2], acc[2 * s + 1][3], ah[3], al[3]);
#pragma unroll
        for (int n = 0; n < 8; n += 2) {
          if (n < nt) {
            unsigned b[4];
            gch_ldsm4t(b, v_s + (s * 16 + (mat & 1) * 8 + (lane & 7)) * (vdim + 8) + n0 + n * 8 + (mat >> 1) * 8);
            gch_mma(y[n], ah, b[0], b[1]);
            gch_mma(y[n + 1], ah, b[2], b[3]);
            gch_mma(y[n], al, b[0], b[1]);
            gch_mma(y[n + 1], al, b[2], b[3]);
          }
        }
      }
    }
    for (int kk = 0; kk < dim; kk += 16) {
      const float* r_lo = rp + (warp * 16 + g) * ks + kk + cp;
      const float2 q0 = *reinterpret_cast<const float2*>(r_lo), q1 = *reinterpret_cast<const float2*>(r_lo + 8 * ks),
                   q2 = *reinterpret_cast<const float2*>(r_lo + 8), q3 = *reinterpret_cast<const float2*>(r_lo + 8 * ks + 8);
      unsigned ah[4], al[4];
      uint2 x0[8], x1[8];  // (rounded pair, pair of rests)
      const float* sp = st + (long long)(n0 + g) * dim + kk + cp;
#pragma unroll
      for (int n = 0; n < 8; ++n)
        if (n < nt) {
          x0[n] = *reinterpret_cast<const uint2*>(sp + (long long)n * 8 * dim);
          x1[n] = *reinterpret_cast<const uint2*>(sp + (long long)n * 8 * dim + 8);
        }
      gch_split(q0.x, q0.y, ah[0], al[0]);
      gch_split(q1.x, q1.y, ah[1], al[1]);
      gch_split(q2.x, q2.y, ah[2], al[2]);
      gch_split(q3.x, q3.y, ah[3], al[3]);
#pragma unroll
      for (int n = 0; n < 8; ++n)
        if (n < nt) {
          gch_mma(y[n], ah, x0[n].x, x1[n].x);
          gch_mma(y[n], ah, x0[n].y, x1[n].y);
          gch_mma(y[n], al, x0[n].x, x1[n].x);
        }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int row = warp * 16 + g + 8 * h;
      if (row >= cn) continue;
      float* dst = out + ((long long)(t0 + row) * heads + head) * vdim + n0 + cp;
#pragma unroll
      for (int n = 0; n < 8; ++n)
        if (n < nt) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(y[n][2 * h], y[n][2 * h + 1]);
    }
  }
}

static size_t gch_fold_smem(int dim, int vdim) {
  return (size_t)(GCH_Q * (dim + 4) + GCH_SUBS * dim) * 4 + (size_t)GCH_Q * (vdim + 8) * 2;
}
static size_t gch_out_smem(int dim, int vdim) {
  return (size_t)(2 * GCH_Q * (dim + 4) + GCH_SUBS * dim + GCH_SUBS * 80) * 4 + (size_t)GCH_Q * (vdim + 8) * 2 +
         (size_t)GCH_Q * (dim + 8) * 2;
}

// Sizes the chunked form takes (bfloat16): key and value sizes that are multiples of 16, as far as the shared memory reaches.
extern "C" int ullm_gla_chunk_supported(int heads, int dim, int vdim) {
  return heads > 0 && heads <= 65535 && dim > 0 && vdim > 0 && dim % 16 == 0 && vdim % 16 == 0 && dim <= GCH_MAX_DIM &&
         gch_out_smem(dim, vdim) <= 227 * 1024;
}
// Chunks a step of `tokens` tokens and `requests` requests has at most; floats of scratch per chunk.
extern "C" int ullm_gla_chunk_tiles(int tokens, int requests) { return tokens / GCH_Q + requests; }
extern "C" long long ullm_gla_chunk_floats(int heads, int dim, int vdim) { return (long long)heads * dim * (vdim + 1); }

template <typename K>
static int gch_allow(K kernel, size_t smem, size_t* have) {
  if (smem > *have) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      cudaGetLastError();
      return ULLM_ERR_LAUNCH;
    }
    cudaFuncSetAttribute(kernel, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
    *have = smem;
  }
  return ULLM_OK;
}

// Arguments as `ullm_gla_recurrence` with `decay` [tokens, heads * dim] the decays themselves; `scratch`:
// ullm_gla_chunk_tiles * ullm_gla_chunk_floats floats.  Runs the requests that bring MORE than `least` tokens and leaves the
// others alone.
extern "C" int ullm_gla_chunk(const void* qkv, long long row_stride, int q_off, int k_off, int v_off, const float* decay,
                              long long decay_stride, const float* bonus, float q_scale, float* scratch, float* state,
                              long long state_stride, const int* cu_q, const int* req_slots, const int* token_req, float* out,
                              int tokens, int requests, int heads, int dim, int vdim, int num_slots, int least, int* status,
                              void* stream) {
  cudaStream_t st = (cudaStream_t)stream;
  if (tokens < 0 || requests < 0 || num_slots <= 0 || scratch == nullptr) return ULLM_ERR_BAD_SIZE;
  if (!ullm_gla_chunk_supported(heads, dim, vdim) || requests > 65535) return ULLM_ERR_UNSUPPORTED;
  if (state_stride < (long long)heads * dim * vdim || state_stride % 4) return ULLM_ERR_BAD_SIZE;
  if (row_stride % 8 || q_off % 8 || k_off % 8 || v_off % 8 || decay_stride % 4 ||
      (((uintptr_t)qkv | (uintptr_t)scratch | (uintptr_t)state | (uintptr_t)decay) & 15) || ((uintptr_t)out & 7))
    return ULLM_ERR_BAD_SIZE;
  if (tokens == 0 || requests == 0) return ULLM_OK;
  const int tiles = ullm_gla_chunk_tiles(tokens, requests);
  float* fold = scratch;
  float* total = scratch + (long long)tiles * heads * dim * vdim;
  static size_t fold_smem = 48 * 1024, out_smem[2] = {48 * 1024, 48 * 1024};
  const size_t fs = gch_fold_smem(dim, vdim), os = gch_out_smem(dim, vdim);
  int rc = gch_allow(gla_fold_kernel, fs, &fold_smem);
  if (rc != ULLM_OK) return rc;
  rc = bonus != nullptr ? gch_allow(gla_out_kernel<true>, os, &out_smem[0]) : gch_allow(gla_out_kernel<false>, os, &out_smem[1]);
  if (rc != ULLM_OK) return rc;
  const dim3 grid(tiles, heads), block(GCH_THREADS);
  rc = ullm_launch_kernel(gla_fold_kernel, grid, block, fs, st, (const __nv_bfloat16*)qkv, row_stride, k_off, v_off, decay,
                          decay_stride, cu_q, token_req, requests, least, heads, dim, vdim, fold, total);
  if (rc != ULLM_OK) return rc;
  rc = ullm_launch_kernel(gla_scan_kernel, dim3((dim * vdim / 2 + 127) / 128, heads, requests), dim3(128), 0, st, fold,
                          (const float*)total, state, state_stride, cu_q, req_slots, token_req, least, heads, dim, vdim,
                          num_slots, status);
  if (rc != ULLM_OK) return rc;
  if (bonus != nullptr)
    return ullm_launch_kernel(gla_out_kernel<true>, grid, block, os, st, (const __nv_bfloat16*)qkv, row_stride, q_off, k_off,
                              v_off, decay, decay_stride, bonus, q_scale, cu_q, token_req, requests, least, heads, dim, vdim,
                              (const float*)fold, out);
  return ullm_launch_kernel(gla_out_kernel<false>, grid, block, os, st, (const __nv_bfloat16*)qkv, row_stride, q_off, k_off,
                            v_off, decay, decay_stride, bonus, q_scale, cu_q, token_req, requests, least, heads, dim, vdim,
                            (const float*)fold, out);
}
