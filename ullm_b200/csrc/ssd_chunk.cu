// The recurrence of csrc/ssd.cu for prompt portions in bfloat16, SSC_Q tokens at a time on the tensor cores.
//
// With a_t the logarithm of the decay, c_t = a_1 + .. + a_t inside a chunk, and S the state in front of the chunk:
//
//   y_t = e^(c_t) C_t^T S + sum_{s <= t} e^(c_t - c_s) dt_s (C_t . B_s) x_s + D x_t
//   S'  = e^(c_Q) S + sum_s B_s (e^(c_Q - c_s) dt_s x_s)^T
//
// so a chunk is four small matrix products instead of SSC_Q dependent steps.  The scores C_t . B_s are the same for all
// heads of a group: `ssd_scores_kernel` forms them once per chunk and group (32-bit).  `ssd_chunk_kernel` walks a request's
// chunks in order; a block owns (request, head, PT columns of S) and keeps its part of S in 32-bit accumulators from chunk
// to chunk; the next chunk's rows arrive by cp.async meanwhile.
//
// Precision: everything is accumulated in 32-bit.  B, C and x are exact bfloat16 operands; the 32-bit operands (the
// weighted scores, the weighted x, the state in the read-out) enter as TWO bfloat16 terms, the rounded value and the rounded
// rest, so that a product keeps 16 bits of them or more, and no chunk ever sees a state rounded to 16 bits.
//
// mma.sync m16n8k16; accumulator and operand fragments as in csrc/attention_window.cu.
#include "common.cuh"

#define SSC_Q 64        // tokens per chunk
#define SSC_THREADS 128
#define SSC_G_STRIDE 72  // floats between rows of a chunk's scores in shared memory (free of bank conflicts)

__device__ __forceinline__ void ssc_cp_async_16(void* smem, const void* gmem, bool pred) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  const int n = pred ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(n));
}
__device__ __forceinline__ void ssc_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N>
__device__ __forceinline__ void ssc_wait() {
  asm volatile("cp.async.wait_group %0;\n" ::"n"(N));
}
__device__ __forceinline__ void ssc_ldsm4(unsigned (&r)[4], const void* p) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(s));
}
__device__ __forceinline__ void ssc_ldsm4t(unsigned (&r)[4], const void* p) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(s));
}
__device__ __forceinline__ void ssc_mma(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (v0, v1) as a pair of rounded values and a pair of rounded rests
__device__ __forceinline__ void ssc_split(float v0, float v1, unsigned& hi, unsigned& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(v0, v1);
  const __nv_bfloat162 l = __floats2bfloat162_rn(v0 - __bfloat162float(h.x), v1 - __bfloat162float(h.y));
  hi = *reinterpret_cast<const unsigned*>(&h);
  lo = *reinterpret_cast<const unsigned*>(&l);
}

// scores[(group * tokens + t) * SSC_Q + s] = C_t . B_s for the tokens s <= t of t's chunk (others: undefined).  Chunks
// are counted from a request's first token of the step; requests of at most `least` tokens are left out.
__global__ void __launch_bounds__(SSC_THREADS)
ssd_scores_kernel(const __nv_bfloat16* __restrict__ xbc, long long row_stride, int b_off, int c_off, int n_state,
                  const int* __restrict__ cu_q, const int* __restrict__ token_req, int requests, int tokens, int least,
                  float* __restrict__ scores) {
  extern __shared__ __align__(16) unsigned char sc_smem[];
  pdl_launch_dependents();
  pdl_wait();
  int tile = blockIdx.x, t0 = 0, cn = 0;
  for (int i = 0; i < requests; ++i) {
    const int b = cu_q[i], n = cu_q[i + 1] - b;
    if (n <= least) continue;
    const int nt = (n + SSC_Q - 1) / SSC_Q;
    if (tile < nt) {
      t0 = b + tile * SSC_Q;
      cn = min(SSC_Q, n - tile * SSC_Q);
      break;
    }
    tile -= nt;
  }
  if (cn == 0 || token_req[t0] < 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, group = blockIdx.y;
  const int rs = n_state * 2 + 16;  // bytes between rows
  unsigned char* c_s = sc_smem;
  unsigned char* b_s = sc_smem + SSC_Q * rs;
  const int pieces = n_state / 8;
  for (int i = tid; i < SSC_Q * pieces; i += SSC_THREADS) {
    const int row = i / pieces, ch = i - row * pieces;
    const bool ok = row < cn;
    const __nv_bfloat16* src = xbc + (long long)(t0 + (ok ? row : 0)) * row_stride + group * n_state + ch * 8;
    ssc_cp_async_16(c_s + row * rs + ch * 16, src + c_off, ok);
    ssc_cp_async_16(b_s + row * rs + ch * 16, src + b_off, ok);
  }
  ssc_commit();
  ssc_wait<0>();
  __syncthreads();
  if (warp * 16 >= cn) return;
  float acc[SSC_Q / 8][4];
#pragma unroll
  for (int j = 0; j < SSC_Q / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  const int mat = lane >> 3;
  const unsigned char* ap = c_s + (warp * 16 + (mat & 1) * 8 + (lane & 7)) * rs + (mat >> 1) * 16;
  const unsigned char* bp = b_s + ((mat >> 1) * 8 + (lane & 7)) * rs + (mat & 1) * 16;
  for (int k = 0; k < n_state / 16; ++k) {
    unsigned a[4];
    ssc_ldsm4(a, ap + k * 32);
#pragma unroll
    for (int j = 0; j < SSC_Q / 8; j += 2) {
      if (j / 2 > warp) continue;  // (above the diagonal)
      unsigned b[4];
      ssc_ldsm4(b, bp + j * 8 * rs + k * 32);
      ssc_mma(acc[j], a, b[0], b[1]);
      ssc_mma(acc[j + 1], a, b[2], b[3]);
    }
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int row = warp * 16 + (lane >> 2) + h * 8;
    if (row >= cn) continue;
    float* dst = scores + ((long long)group * tokens + t0 + row) * SSC_Q + (lane & 3) * 2;
#pragma unroll
    for (int j = 0; j < SSC_Q / 8; ++j)
      if (j / 2 <= warp) *reinterpret_cast<float2*>(dst + j * 8) = make_float2(acc[j][2 * h], acc[j][2 * h + 1]);
  }
}

// PT: columns of S a block owns (16 or 32); n_state = 32 * NT.  Two sets of four warps work on a chunk side by side: set 0
// forms its y (warp w the rows 16 w .. 16 w + 15) from the state in front of it, which waits in shared memory as two bfloat16
// terms; set 1 keeps S^T [PT][N] in accumulators (warp w the columns w N / 4 ..), adds the chunk to it, and fetches the next
// chunk's rows and decays meanwhile.  SB: buffers of the state's terms (with two, one barrier of the block per chunk; with
// one, where two do not fit, a second barrier stands in front of their renewal).
template <int PT, int NT, int SB>
__global__ void __launch_bounds__(2 * SSC_THREADS)
ssd_chunk_kernel(const __nv_bfloat16* __restrict__ xbc, long long row_stride, int b_off, int c_off,
                 const float* __restrict__ dt, const float* __restrict__ log_decay, const float* __restrict__ d_skip,
                 const float* __restrict__ scores, float* __restrict__ state, long long state_stride,
                 const int* __restrict__ cu_q, const int* __restrict__ req_slots, const int* __restrict__ token_req,
                 float* __restrict__ out, int heads, int pdim, int per_group, int tokens, int num_slots, int least,
                 int* status, long long dt_stride) {
  constexpr int N = 32 * NT, NW = N / 4;      // a warp's columns of S^T
  constexpr int RS = N * 2 + 16;              // bytes between rows of B, C and S
  constexpr int XS = PT * 2 + 16;             // ... of x
  constexpr int BC = SSC_Q * RS, XB = SSC_Q * XS, GB = SSC_Q * SSC_G_STRIDE * 4;
  constexpr int STAGE = 2 * BC + XB + GB, ST = PT * RS;
  constexpr int MT = PT / 16, PN = PT / 8;
  extern __shared__ __align__(16) unsigned char sc_smem[];
  __shared__ float s_cum[2][SSC_Q], s_dt[2][SSC_Q], s_e[2][SSC_Q], s_w[2][SSC_Q];
  __shared__ float s_total[2];
  pdl_launch_dependents();
  pdl_wait();
  const int req = blockIdx.z, head = blockIdx.y, p0 = blockIdx.x * PT;
  const int t0 = cu_q[req], n = cu_q[req + 1] - t0;
  if (n <= least || token_req[t0] < 0) return;
  const int slot = req_slots[req];
  const int tid = threadIdx.x & (SSC_THREADS - 1), warp = tid >> 5, lane = tid & 31;
  const bool keeper = threadIdx.x >= SSC_THREADS;  // set 1
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0) ullm_report(status, ULLM_STATUS_SLOT, req, slot);
    return;
  }
  const int group = head / per_group;
  unsigned char* s_terms = sc_smem + 2 * STAGE;  // [SB]: S^T rounded [PT][N], then the rests
  unsigned char* xh_s = s_terms + SB * 2 * ST;   // weighted x rounded, [SSC_Q][PT]
  unsigned char* xl_s = xh_s + XB;
  const int mat = lane >> 3;
  const int chunks = (n + SSC_Q - 1) / SSC_Q;

  if (!keeper) {
    const float skip = d_skip[head];
    __syncthreads();  // chunk 0, its decays and the first state's terms are there
    for (int c = 0; c < chunks; ++c) {
      const int cn = min(SSC_Q, n - c * SSC_Q), cb = c & 1;
      const unsigned char* stg = sc_smem + cb * STAGE;
      const unsigned char* sh_s = s_terms + (SB == 2 ? cb : 0) * 2 * ST;
      const unsigned char* sl_s = sh_s + ST;
      const unsigned char* x_s = stg + 2 * BC;
      const int tr = warp * 16;  // the warp's rows of y
      if (tr < cn) {
        float y[PN][4], yi[PN][4];
#pragma unroll
        for (int j = 0; j < PN; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) y[j][e] = yi[j][e] = 0.f;
        // what the state in front of the chunk gives
#pragma unroll(4)
        for (int k = 0; k < N / 16; ++k) {
          unsigned a[4];
          ssc_ldsm4(a, stg + (tr + (mat & 1) * 8 + (lane & 7)) * RS + (k * 16 + (mat >> 1) * 8) * 2);
#pragma unroll
          for (int j = 0; j < PN; j += 2) {
            const int off = (j * 8 + (mat >> 1) * 8 + (lane & 7)) * RS + (k * 16 + (mat & 1) * 8) * 2;
            unsigned bh[4], bl[4];
            ssc_ldsm4(bh, sh_s + off);
            ssc_ldsm4(bl, sl_s + off);
            ssc_mma(yi[j], a, bh[0], bh[1]);
            ssc_mma(yi[j + 1], a, bh[2], bh[3]);
            ssc_mma(yi[j], a, bl[0], bl[1]);
            ssc_mma(yi[j + 1], a, bl[2], bl[3]);
          }
        }
        // what the tokens of this chunk leave to one another
        const float* g_s = reinterpret_cast<const float*>(stg + 2 * BC + XB);
        const int r0 = tr + (lane >> 2);
        const float cr[2] = {s_cum[cb][r0], s_cum[cb][r0 + 8]};
#pragma unroll
        for (int ks = 0; ks < SSC_Q / 16; ++ks) {
          if (ks > warp) continue;
          unsigned ah[4], al[4];
#pragma unroll
          for (int q = 0; q < 4; ++q) {  // the fragment's four register pairs: rows + 8 (q & 1), columns + 8 (q >> 1)
            const int row = r0 + (q & 1) * 8, s = ks * 16 + (q >> 1) * 8 + (lane & 3) * 2;
            const float2 g = *reinterpret_cast<const float2*>(g_s + row * SSC_G_STRIDE + s);
            const float2 cs = *reinterpret_cast<const float2*>(&s_cum[cb][s]);
            const float2 ds = *reinterpret_cast<const float2*>(&s_dt[cb][s]);
            const float v0 = s <= row ? g.x * (__expf(cr[q & 1] - cs.x) * ds.x) : 0.f;
            const float v1 = s + 1 <= row ? g.y * (__expf(cr[q & 1] - cs.y) * ds.y) : 0.f;
            ssc_split(v0, v1, ah[q], al[q]);
          }
#pragma unroll
          for (int j = 0; j < PN; j += 2) {
            unsigned b[4];
            ssc_ldsm4t(b, x_s + (ks * 16 + (mat & 1) * 8 + (lane & 7)) * XS + (j * 8 + (mat >> 1) * 8) * 2);
            ssc_mma(y[j], ah, b[0], b[1]);
            ssc_mma(y[j + 1], ah, b[2], b[3]);
            ssc_mma(y[j], al, b[0], b[1]);
            ssc_mma(y[j + 1], al, b[2], b[3]);
          }
        }
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int row = r0 + 8 * h;
          if (row >= cn) continue;
          const float e = s_e[cb][row];
          float* dst = out + ((long long)(t0 + c * SSC_Q + row) * heads + head) * pdim + p0 + (lane & 3) * 2;
#pragma unroll
          for (int j = 0; j < PN; ++j) {
            const __nv_bfloat162 xv =
                *reinterpret_cast<const __nv_bfloat162*>(x_s + row * XS + (j * 8 + (lane & 3) * 2) * 2);
            *reinterpret_cast<float2*>(dst + j * 8) =
                make_float2(fmaf(e, yi[j][2 * h], y[j][2 * h]) + skip * __bfloat162float(xv.x),
                            fmaf(e, yi[j][2 * h + 1], y[j][2 * h + 1]) + skip * __bfloat162float(xv.y));
          }
        }
      }
      if (SB == 1) __syncthreads();  // the state's terms have been read
      __syncthreads();               // the chunk is done, the next one is there
    }
    return;
  }

  auto issue = [&](int chunk) {
    unsigned char* st = sc_smem + (chunk & 1) * STAGE;
    const int c0 = t0 + chunk * SSC_Q, cn = min(SSC_Q, n - chunk * SSC_Q);
    constexpr int PIECES = N / 8, XP = PT / 8, GP = SSC_Q / 4;
    for (int i = tid; i < SSC_Q * PIECES; i += SSC_THREADS) {
      const int row = i / PIECES, ch = i - row * PIECES;
      const bool ok = row < cn;
      const __nv_bfloat16* src = xbc + (long long)(c0 + (ok ? row : 0)) * row_stride + group * N + ch * 8;
      ssc_cp_async_16(st + row * RS + ch * 16, src + c_off, ok);
      ssc_cp_async_16(st + BC + row * RS + ch * 16, src + b_off, ok);
    }
    for (int i = tid; i < SSC_Q * XP; i += SSC_THREADS) {
      const int row = i / XP, ch = i - row * XP;
      const bool ok = row < cn;
      ssc_cp_async_16(st + 2 * BC + row * XS + ch * 16,
                      xbc + (long long)(c0 + (ok ? row : 0)) * row_stride + head * pdim + p0 + ch * 8, ok);
    }
    for (int i = tid; i < SSC_Q * GP; i += SSC_THREADS) {
      const int row = i / GP, ch = i - row * GP;
      // (only what lies on or below the diagonal's 16 x 16 blocks was written)
      const bool ok = row < cn && (ch >> 2) <= (row >> 4);
      ssc_cp_async_16(st + 2 * BC + XB + row * (SSC_G_STRIDE * 4) + ch * 16,
                      scores + ((long long)group * tokens + c0 + (ok ? row : 0)) * SSC_Q + ch * 4, ok);
    }
    ssc_commit();
  };
  float pa[2] = {0.f, 0.f}, pd[2] = {0.f, 0.f};  // warp 0: decays and steps of tokens 2 lane, 2 lane + 1, a chunk ahead
  auto fetch = [&](int chunk) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = chunk * SSC_Q + 2 * lane + i;
      pa[i] = t < n ? log_decay[(long long)(t0 + t) * dt_stride + head] : 0.f;
      pd[i] = t < n ? dt[(long long)(t0 + t) * dt_stride + head] : 0.f;
    }
  };
  auto weigh = [&](int buf) {  // warp 0: the chunk's running sums and weights from what `fetch` brought
    float run = pa[0] + pa[1];  // the inclusive sum over the lanes
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += v;
    }
    const float total = __shfl_sync(0xffffffffu, run, 31);
    const float cu[2] = {run - pa[1], run};
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      s_cum[buf][2 * lane + i] = cu[i];
      s_dt[buf][2 * lane + i] = pd[i];
      s_e[buf][2 * lane + i] = expf(cu[i]);
      s_w[buf][2 * lane + i] = expf(total - cu[i]) * pd[i];
    }
    if (lane == 0) s_total[buf] = expf(total);
  };

  // S^T fragments: rows p = 16 m + lane / 4 (+ 8), columns n = warp * NW + 8 j + 2 (lane % 4) (+ 1)
  float S[MT][NT][4];
  auto put_terms = [&](int buf) {
    unsigned char* sh_s = s_terms + (SB == 2 ? buf : 0) * 2 * ST;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          unsigned hi, lo;
          ssc_split(S[m][j][2 * h], S[m][j][2 * h + 1], hi, lo);
          const int off = (16 * m + (lane >> 2) + 8 * h) * RS + (warp * NW + 8 * j + (lane & 3) * 2) * 2;
          *reinterpret_cast<unsigned*>(sh_s + off) = hi;
          *reinterpret_cast<unsigned*>(sh_s + ST + off) = lo;
        }
  };
  issue(0);
  float* st_head = state + (long long)slot * state_stride + ((long long)head * pdim + p0) * N;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const float2 v = *reinterpret_cast<const float2*>(st_head + (long long)(16 * m + (lane >> 2) + 8 * h) * N +
                                                          warp * NW + 8 * j + (lane & 3) * 2);
        S[m][j][2 * h] = v.x;
        S[m][j][2 * h + 1] = v.y;
      }
  if (warp == 0) {
    fetch(0);
    weigh(0);
    if (chunks > 1) fetch(1);
  }
  put_terms(0);
  ssc_wait<0>();
  __syncthreads();
  for (int c = 0; c < chunks; ++c) {
    const int cb = c & 1;
    unsigned char* stg = sc_smem + cb * STAGE;
    if (c + 1 < chunks) issue(c + 1);
    // x weighted by its step and by what is left of it at the chunk's end, as two terms
    const unsigned char* x_s = stg + 2 * BC;
    for (int i = tid; i < SSC_Q * PT / 2; i += SSC_THREADS) {
      const int row = i / (PT / 2), q = i - row * (PT / 2);
      const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(x_s + row * XS + q * 4);
      const float w = s_w[cb][row];
      unsigned hi, lo;
      ssc_split(__bfloat162float(v.x) * w, __bfloat162float(v.y) * w, hi, lo);
      *reinterpret_cast<unsigned*>(xh_s + row * XS + q * 4) = hi;
      *reinterpret_cast<unsigned*>(xl_s + row * XS + q * 4) = lo;
    }
    asm volatile("bar.sync 1, %0;" ::"n"(SSC_THREADS) : "memory");  // (set 1 alone)
    const float total = s_total[cb];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[m][j][e] *= total;
#pragma unroll
    for (int ks = 0; ks < SSC_Q / 16; ++ks) {
      unsigned ah[MT][4], al[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const int off = (ks * 16 + (mat >> 1) * 8 + (lane & 7)) * XS + (16 * m + (mat & 1) * 8) * 2;
        ssc_ldsm4t(ah[m], xh_s + off);
        ssc_ldsm4t(al[m], xl_s + off);
      }
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        // (with one tile per warp the second half of the load is the next warp's, or the row's padding: unused)
        unsigned b[4];
        ssc_ldsm4t(b, stg + BC + (ks * 16 + (mat & 1) * 8 + (lane & 7)) * RS + (warp * NW + j * 8 + (mat >> 1) * 8) * 2);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          ssc_mma(S[m][j], ah[m], b[0], b[1]);
          if (NT > 1) ssc_mma(S[m][NT > 1 ? j + 1 : j], ah[m], b[2], b[3]);
          ssc_mma(S[m][j], al[m], b[0], b[1]);
          if (NT > 1) ssc_mma(S[m][NT > 1 ? j + 1 : j], al[m], b[2], b[3]);
        }
      }
    }
    if (SB == 1) __syncthreads();  // set 0 has read the state's terms
    if (c + 1 < chunks) {
      put_terms(cb ^ 1);
      if (warp == 0) {
        weigh(cb ^ 1);
        if (c + 2 < chunks) fetch(c + 2);
      }
      ssc_wait<0>();
    }
    __syncthreads();
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int h = 0; h < 2; ++h)
        *reinterpret_cast<float2*>(st_head + (long long)(16 * m + (lane >> 2) + 8 * h) * N + warp * NW + 8 * j +
                                   (lane & 3) * 2) = make_float2(S[m][j][2 * h], S[m][j][2 * h + 1]);
}

// Sizes the chunked form takes (bfloat16): states of 32, 64, 128 or 256 rows, columns a multiple of 16.
extern "C" int ullm_ssd_chunk_supported(int heads, int n_state, int pdim, int groups) {
  return heads > 0 && groups > 0 && heads % groups == 0 && heads <= 65535 && pdim > 0 && pdim % 16 == 0 &&
         (n_state == 32 || n_state == 64 || n_state == 128 || n_state == 256);
}
extern "C" int ullm_ssd_chunk_tokens(void) { return SSC_Q; }

template <int PT, int NT>
static int chunk_go(const void* xbc, long long row_stride, int b_off, int c_off, const float* dt, const float* log_decay,
                    const float* d_skip, const float* scores, float* state, long long state_stride, const int* cu_q,
                    const int* req_slots, const int* token_req, float* out, int tokens, int requests, int heads, int pdim,
                    int groups, int num_slots, int least, int* status, long long dt_stride, cudaStream_t st) {
  constexpr int N = 32 * NT, RS = N * 2 + 16, XS = PT * 2 + 16;
  constexpr size_t stages = 2 * (2 * SSC_Q * RS + SSC_Q * XS + SSC_Q * SSC_G_STRIDE * 4) + 2 * SSC_Q * XS;
  constexpr int SB = stages + 4 * PT * RS + 2304 <= 227 * 1024 ? 2 : 1;  // (2304: more than the static arrays)
  constexpr size_t smem = stages + SB * 2 * PT * RS;
  static_assert(smem + 2304 <= 227 * 1024, "a chunk's stages fit the shared memory");
  static int attr_set = 0;
  if (!attr_set) {
    if (cudaFuncSetAttribute(ssd_chunk_kernel<PT, NT, SB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      cudaGetLastError();
      return ULLM_ERR_LAUNCH;
    }
    cudaFuncSetAttribute(ssd_chunk_kernel<PT, NT, SB>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
    attr_set = 1;
  }
  return ullm_launch_kernel(ssd_chunk_kernel<PT, NT, SB>, dim3(pdim / PT, heads, requests), dim3(2 * SSC_THREADS), smem, st,
                            (const __nv_bfloat16*)xbc, row_stride, b_off, c_off, dt, log_decay, d_skip, scores, state,
                            state_stride, cu_q, req_slots, token_req, out, heads, pdim, heads / groups, tokens, num_slots,
                            least, status, dt_stride);
}

// Arguments as `ullm_ssd_recurrence`; `scores`: scratch of groups * tokens * SSC_Q floats.  Runs the requests that bring
// MORE than `least` tokens and leaves the others alone.
extern "C" int ullm_ssd_chunk(const void* xbc, long long row_stride, int b_off, int c_off, const float* dt,
                              const float* log_decay, const float* d_skip, float* scores, float* state,
                              long long state_stride, const int* cu_q, const int* req_slots, const int* token_req, float* out,
                              int tokens, int requests, int heads, int n_state, int pdim, int groups, int num_slots,
                              int least, int* status, void* stream, long long dt_stride) {
  cudaStream_t st = (cudaStream_t)stream;
  if (tokens < 0 || requests < 0 || num_slots <= 0 || scores == nullptr) return ULLM_ERR_BAD_SIZE;
  if (!ullm_ssd_chunk_supported(heads, n_state, pdim, groups) || requests > 65535 || groups > 65535) return ULLM_ERR_UNSUPPORTED;
  if (state_stride < (long long)heads * pdim * n_state || state_stride % 2) return ULLM_ERR_BAD_SIZE;
  if (row_stride % 8 || b_off % 8 || c_off % 8 || (((uintptr_t)xbc | (uintptr_t)scores) & 15) || (((uintptr_t)state | (uintptr_t)out) & 7))
    return ULLM_ERR_BAD_SIZE;
  if (tokens == 0 || requests == 0) return ULLM_OK;
  const int tiles = tokens / SSC_Q + requests;  // an upper bound on the chunks, however the tokens are spread
  const size_t sc_smem = (size_t)2 * SSC_Q * (n_state * 2 + 16);
  static size_t attr_smem = 48 * 1024;
  if (sc_smem > attr_smem) {
    if (cudaFuncSetAttribute(ssd_scores_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sc_smem) != cudaSuccess) {
      cudaGetLastError();
      return ULLM_ERR_LAUNCH;
    }
    attr_smem = sc_smem;
  }
  const int rc = ullm_launch_kernel(ssd_scores_kernel, dim3(tiles, groups), dim3(SSC_THREADS), sc_smem, st,
                                    (const __nv_bfloat16*)xbc, row_stride, b_off, c_off, n_state, cu_q, token_req, requests,
                                    tokens, least, scores);
  if (rc != ULLM_OK) return rc;
  int sms = 148, dev = 0;
  if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  // 16 or 32 columns per block, by (waves of blocks) x (a chunk's cost, which grows slowly with the columns)
  const int per_sm = n_state <= 64 ? 3 : (n_state == 128 ? 2 : 1);
  const long long b16 = (long long)(pdim / 16) * heads * requests, b32 = (long long)(pdim / 32) * heads * requests;
  const double places = (double)per_sm * sms;
  const double c16 = b16 <= sms ? 1.0 : (double)((long long)((b16 + places - 1) / places)) * per_sm;
  const double c32 = (b32 <= sms ? 1.0 : (double)((long long)((b32 + places - 1) / places)) * per_sm) * 1.5;
  const bool wide = pdim % 32 == 0 && c32 < c16;
#define SSC_GO(PT, NT)                                                                                               \
  return chunk_go<PT, NT>(xbc, row_stride, b_off, c_off, dt, log_decay, d_skip, scores, state, state_stride, cu_q,    \
                          req_slots, token_req, out, tokens, requests, heads, pdim, groups, num_slots, least, status, dt_stride, st)
  switch (n_state) {
    case 32:
      if (wide) SSC_GO(32, 1);
      SSC_GO(16, 1);
    case 64:
      if (wide) SSC_GO(32, 2);
      SSC_GO(16, 2);
    case 128:
      if (wide) SSC_GO(32, 4);
      SSC_GO(16, 4);
    default:
      if (wide) SSC_GO(32, 8);
      SSC_GO(16, 8);
  }
#undef SSC_GO
}
