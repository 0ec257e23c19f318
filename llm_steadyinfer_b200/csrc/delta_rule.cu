// The gated delta rule: a linear-attention recurrence whose state is a matrix per head that forgets by a scalar
// decay and is corrected, not just added to, by each token:
//   S <- g_t S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t          S is dk x dv, fp32
// so the read-out sees the token's own write. Everything that enters the recurrence is fp32.
//
// Two kernels. `delta_prepare` works on all rows at once: it makes q and k unit vectors per head
// (x / sqrt(sum(x^2) + 1e-6), q also times `q_scale`), beta = sigmoid(b), g = exp(-exp(A_log) * softplus(a + dt_bias))
// and q . k of the prepared vectors.
// `delta_scan` walks the tokens of every sequence of the step in order. The columns of S are independent of one
// another, so a block takes (sequence, head, a cut of the columns); thread (column j, part p) keeps RPT neighbouring
// rows of column j in registers. Per token it forms its parts of k . S[:, j] and q . S[:, j] from the old state (two
// rows at a time on the packed fp32 instructions, two sums each, so that the chain of dependent additions is short),
// the NP parts of a column (neighbouring lanes) are added with shuffles, and then
//   kS = g (k . S_old[:, j]);  u_j = beta (v_j - kS);  o_j = g (q . S_old[:, j]) + (q . k) u_j;  S[:, j] <- g S_old[:, j] + k u_j
// which is the order above with one pass over the registers for the sums and one for the update. q, k, v, beta, g and
// q . k of CHUNK tokens arrive by cp.async in the half of shared memory that is not being computed on; within a chunk
// the warps do not wait for one another.
// A request's state lies at the start of its slot, head by head, each head as [RPT][dv][NP] (see delta_shape); a
// portion that begins at position 0 starts from zero whatever the slot held.
//
// With a decay per key channel (a factor for every row of S) the same recurrence runs in `channel_delta_scan`: S <- diag(g_t) S
// first, then the sums over the decayed state, four packed operations for two rows as before. `channel_delta_prepare` makes
// the decays, beta and q . k; q and k arrive as unit vectors.
#include "common.cuh"
#include <math.h>

__device__ __forceinline__ float softplus_d(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// xc: fp32 rows [q: G*dk | k: G*dk | ...] (the convolution's output), normalised in place.
// ba: rows of the projection holding b (H values at b_off) and a (H values at a_off) in the compute dtype.
// bg: fp32 [T, 2H + G]: beta, then g, then q . k of the prepared vectors per query/key head.
template <typename T>
__global__ void __launch_bounds__(128) delta_prepare_kernel(float* __restrict__ xc, long long xc_stride, const T* __restrict__ ba,
    long long ba_stride, int b_off, int a_off, const float* __restrict__ a_log, const float* __restrict__ dt_bias,
    float* __restrict__ bg, int G, int H, int dk, float q_scale) {
  pdl_prologue();
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  float* row = xc + (size_t)t * xc_stride;
  float* bgr = bg + (size_t)t * (2 * H + G);
  for (int gh = warp; gh < G; gh += nwarps) {          // a warp takes the query and the key of one head
    float* q = row + (size_t)gh * dk;
    float* k = row + (size_t)(G + gh) * dk;
    float sq = 0.f, sk = 0.f;
    for (int i = lane; i < dk; i += 32) { sq += q[i] * q[i]; sk += k[i] * k[i]; }
    const float fq = rsqrtf(warp_sum(sq) + 1e-6f) * q_scale, fk = rsqrtf(warp_sum(sk) + 1e-6f);
    float dot = 0.f;
    for (int i = lane; i < dk; i += 32) {
      const float a = q[i] * fq, b = k[i] * fk;
      q[i] = a; k[i] = b;
      dot = fmaf(a, b, dot);
    }
    dot = warp_sum(dot);
    if (lane == 0) bgr[2 * H + gh] = dot;
  }
  const T* r = ba + (size_t)t * ba_stride;
  for (int h = threadIdx.x; h < H; h += blockDim.x) {
    bgr[h] = 1.f / (1.f + expf(-to_f32<T>(r[b_off + h])));
    bgr[H + h] = expf(-expf(a_log[h]) * softplus_d(to_f32<T>(r[a_off + h]) + dt_bias[h]));
  }
}

SI_EXPORT int si_delta_prepare(float* xc, long long xc_stride, const void* ba, int dtype, long long ba_stride, int b_off,
                               int a_off, const float* a_log, const float* dt_bias, float* bg, int num_tokens, int G, int H,
                               int dk, float q_scale, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (dtype == SI_BF16)
    si_launch(delta_prepare_kernel<__nv_bfloat16>, dim3(num_tokens), dim3(128), 0, stream, xc, xc_stride,
              (const __nv_bfloat16*)ba, ba_stride, b_off, a_off, a_log, dt_bias, bg, G, H, dk, q_scale);
  else
    si_launch(delta_prepare_kernel<float>, dim3(num_tokens), dim3(128), 0, stream, xc, xc_stride, (const float*)ba,
              ba_stride, b_off, a_off, a_log, dt_bias, bg, G, H, dk, q_scale);
  return si_last_error();
}

#define DELTA_CHUNK 32

__device__ __forceinline__ void delta_cp4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void delta_cp16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src));
}

// The shape for a state of dk x dv: rows a thread (RPT, a multiple of 4) and parts a column (NP, a power of two up to 32,
// RPT * NP >= dk): about sixteen parts. A sequence's tokens are a chain of dependent steps; few rows a thread shorten the
// chain and give a multiprocessor warps to choose from, many parts cost shuffles (measured at 128 x 128, 16 heads, one
// sequence of 2,048 tokens: 16 rows in 8 parts 1.54 ms, 4 rows in 32 parts 0.69 ms).
// Thread (column j, part p) keeps, for c < RPT / 4, the four rows (c * NP + p) * 4 .. + 3 of column j (so that the parts
// read neighbouring 16-byte words of q and k). A head's state lies in the slot as [RPT][dv][NP]: entry
// ((r * dv + j) * NP + p) is the thread's r-th row, so that a block reads and writes whole lines whatever cut of the
// columns it has.
struct DeltaShape { int rpt, np; };
static DeltaShape delta_shape(int dk) {
  DeltaShape s;
  s.rpt = ((dk + 15) / 16 + 3) / 4 * 4;
  int parts = 1;
  while (parts * s.rpt < dk) parts *= 2;
  s.np = parts;
  return s;
}
// fp32 entries of one head's state in a slot
SI_EXPORT long long si_delta_state_floats(int dk, int dv) {
  if (dk <= 0 || dv <= 0 || dk > 512) return -1;
  const DeltaShape s = delta_shape(dk);
  return (long long)s.rpt * s.np * dv;
}

// RPT: rows of a column that a thread keeps, as RPT / 2 pairs (the sums and the update run two rows at a time on the
// packed fp32 instructions). Shared memory: two buffers of CHUNK tokens of [q: RPT * NP | k: RPT * NP | v: cols |
// beta, g, q . k, -] (rows beyond dk stay zero), filled by cp.async one chunk ahead of the sums.
template <int RPT, int NP>
__global__ void __launch_bounds__(256) delta_scan_kernel(const float* __restrict__ xc, long long xc_stride,
    const float* __restrict__ bg, int bg_width, float* __restrict__ state, long long state_stride, float* __restrict__ y,
    long long y_stride, const int* __restrict__ q_start, const int* __restrict__ ctx_len, const int* __restrict__ slots,
    int G, int H, int dk, int dv, int cols) {
  extern __shared__ __align__(16) float sm[];
  pdl_prologue();
  const int s = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * cols;
  const int row0 = q_start[s], n = q_start[s + 1] - row0;
  if (n <= 0) return;
  const int pos0 = ctx_len[s] - n;
  const int g = h / (H / G);
  const int p = threadIdx.x % NP, jl = threadIdx.x / NP;
  const int j = j0 + jl;
  const bool col_ok = jl < cols && j < dv;
  float* S = state + (size_t)slots[s] * state_stride + (size_t)h * RPT * NP * dv + (size_t)(col_ok ? j : 0) * NP + p;
  const size_t s_step = (size_t)dv * NP;
  float2 st[RPT / 2];
#pragma unroll
  for (int r = 0; r < RPT / 2; ++r) {
    st[r].x = (col_ok && pos0 > 0) ? S[(size_t)(2 * r) * s_step] : 0.f;
    st[r].y = (col_ok && pos0 > 0) ? S[(size_t)(2 * r + 1) * s_step] : 0.f;
  }
  const int dkp = RPT * NP;
  const int per_tok = 2 * dkp + ((cols + 3) & ~3) + 4;
  for (int idx = threadIdx.x; idx < 2 * DELTA_CHUNK * per_tok; idx += blockDim.x) sm[idx] = 0.f;
  __syncthreads();
  const size_t q_off = (size_t)g * dk, k_off = (size_t)(G + g) * dk, v_off = (size_t)2 * G * dk + (size_t)h * dv + j0;
  const bool wide = dk % 4 == 0 && xc_stride % 4 == 0 && ((uintptr_t)xc & 15) == 0;      // q and k rows in 16-byte pieces
  // a warp fetches whole tokens (every nwarps-th of the chunk): the copies' bookkeeping is then paid once a token by one
  // warp, not by every warp
  const int unit = wide ? 4 : 1, pieces = 2 * dk / unit, per_half = dk / unit;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  auto fetch = [&](int c0, int buf) {
    const int cn = min(DELTA_CHUNK, n - c0);
    for (int tt = warp; tt < cn; tt += nwarps) {
      float* dst = sm + ((size_t)buf * DELTA_CHUNK + tt) * per_tok;
      const float* row = xc + (size_t)(row0 + c0 + tt) * xc_stride;
      const float* bgr = bg + (size_t)(row0 + c0 + tt) * bg_width;
      for (int t = lane; t < pieces; t += 32) {
        const bool is_q = t < per_half;
        const int i = (is_q ? t : t - per_half) * unit;
        if (wide) delta_cp16(dst + (is_q ? 0 : dkp) + i, row + (is_q ? q_off : k_off) + i);
        else delta_cp4(dst + (is_q ? 0 : dkp) + i, row + (is_q ? q_off : k_off) + i);
      }
      for (int e = lane; e < cols + 3; e += 32) {
        if (e < cols) {
          if (j0 + e < dv) delta_cp4(dst + 2 * dkp + e, row + v_off + e);
        } else {                                     // beta, g, q . k of this head
          const int w = e - cols;
          delta_cp4(dst + per_tok - 4 + w, bgr + (w == 0 ? h : w == 1 ? H + h : 2 * H + g));
        }
      }
    }
    asm volatile("cp.async.commit_group;\n" ::);
  };
  fetch(0, 0);
  int buf = 0;
  for (int c0 = 0; c0 < n; c0 += DELTA_CHUNK, buf ^= 1) {
    const int cn = min(DELTA_CHUNK, n - c0);
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();                            // this chunk has arrived, and everyone is done with the other buffer
    if (c0 + DELTA_CHUNK < n) fetch(c0 + DELTA_CHUNK, buf ^ 1);
    const float* tok = sm + (size_t)buf * DELTA_CHUNK * per_tok;
    float* yp = y + (size_t)(row0 + c0) * y_stride + (size_t)h * dv + j;
#pragma unroll 2
    for (int tt = 0; tt < cn; ++tt, tok += per_tok, yp += y_stride) {
      const float4* q4 = reinterpret_cast<const float4*>(tok) + p;
      const float4* k4 = reinterpret_cast<const float4*>(tok + dkp) + p;
      float2 kk[RPT / 2];
      float2 sk0 = make_float2(0.f, 0.f), sq0 = sk0;
#pragma unroll
      for (int c = 0; c < RPT / 4; ++c) {
        const float4 kv = k4[c * NP], qv = q4[c * NP];
        kk[2 * c] = make_float2(kv.x, kv.y);
        kk[2 * c + 1] = make_float2(kv.z, kv.w);
        sk0 = __ffma2_rn(kk[2 * c], st[2 * c], sk0);
        sq0 = __ffma2_rn(make_float2(qv.x, qv.y), st[2 * c], sq0);
        sk0 = __ffma2_rn(kk[2 * c + 1], st[2 * c + 1], sk0);
        sq0 = __ffma2_rn(make_float2(qv.z, qv.w), st[2 * c + 1], sq0);
      }
      float sk = sk0.x + sk0.y, sq = sq0.x + sq0.y;
#pragma unroll
      for (int o = 1; o < NP; o <<= 1) {
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
      }
      const float4 sc = *reinterpret_cast<const float4*>(tok + per_tok - 4);      // beta, g, q . k
      const float vj = col_ok ? tok[2 * dkp + jl] : 0.f;
      const float u = sc.x * (vj - sc.y * sk);
      const float2 u2 = make_float2(u, u), g2 = make_float2(sc.y, sc.y);
#pragma unroll
      for (int r = 0; r < RPT / 2; ++r) st[r] = __ffma2_rn(kk[r], u2, __fmul2_rn(g2, st[r]));
      if (p == 0 && col_ok) *yp = fmaf(sc.z, u, sc.y * sq);
    }
  }
  if (col_ok) {
#pragma unroll
    for (int r = 0; r < RPT / 2; ++r) {
      S[(size_t)(2 * r) * s_step] = st[r].x;
      S[(size_t)(2 * r + 1) * s_step] = st[r].y;
    }
  }
}

SI_EXPORT int si_delta_scan(const float* xc, long long xc_stride, const float* bg, int bg_width, float* state,
                            long long state_stride, float* y, long long y_stride, const int* q_start, const int* ctx_len,
                            const int* slots, int num_seqs, int G, int H, int dk, int dv, cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (G <= 0 || H % G || dk <= 0 || dv <= 0 || dk > 512 || H > 65535 || bg_width < 2 * H + G) return -2;
  const DeltaShape sh = delta_shape(dk);
  if (sh.rpt * sh.np < dk) return -2;
  if (state_stride < (long long)H * sh.rpt * sh.np * dv) return -2;
  // columns a block: as many as 256 threads hold, fewer while the blocks do not fill the device (a block's tokens are a
  // chain of dependent steps, so more blocks of fewer columns finish sooner); never less than a warp
  int cols = 256 / sh.np;
  if (cols > dv) cols = dv;
  if (cols < 1) cols = 1;
  const long long per = (long long)num_seqs * H;
  while (cols > 1 && (cols / 2) * sh.np >= 32 && per * ((dv + cols - 1) / cols) < si_sm_count()) cols /= 2;
  const int zb = (dv + cols - 1) / cols;
  if (zb > 65535) return -2;
  const int threads = ((cols * sh.np + 31) / 32) * 32;
  const size_t smem = (size_t)2 * DELTA_CHUNK * (2 * sh.np * sh.rpt + ((cols + 3) & ~3) + 4) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  const dim3 grid(num_seqs, H, zb), block(threads);
#define DELTA_LAUNCH(R, P)                                                                                           \
  {                                                                                                                  \
    static size_t configured = 0;                                                                                    \
    if (smem > 48 * 1024 && smem > configured) {                                                                     \
      if (cudaFuncSetAttribute(delta_scan_kernel<R, P>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) \
        return -2;                                                                                                   \
      configured = smem;                                                                                             \
    }                                                                                                                \
    si_launch(delta_scan_kernel<R, P>, grid, block, smem, stream, xc, xc_stride, bg, bg_width, state, state_stride, y, \
              y_stride, q_start, ctx_len, slots, G, H, dk, dv, cols);                                                \
  }
  // (rows a thread, parts a column) as delta_shape gives them: four rows in 1 to 16 parts up to dk = 64, then 16 parts
  if (sh.np < 16) {
    if (sh.rpt != 4) return -2;
    switch (sh.np) {
      case 1: DELTA_LAUNCH(4, 1) break;
      case 2: DELTA_LAUNCH(4, 2) break;
      case 4: DELTA_LAUNCH(4, 4) break;
      case 8: DELTA_LAUNCH(4, 8) break;
      default: return -2;
    }
  } else if (sh.np == 16) {
    switch (sh.rpt) {                        // dk up to 512: up to 32 rows a thread
      case 4: DELTA_LAUNCH(4, 16) break;
      case 8: DELTA_LAUNCH(8, 16) break;
      case 12: DELTA_LAUNCH(12, 16) break;
      case 16: DELTA_LAUNCH(16, 16) break;
      case 20: DELTA_LAUNCH(20, 16) break;
      case 24: DELTA_LAUNCH(24, 16) break;
      case 28: DELTA_LAUNCH(28, 16) break;
      case 32: DELTA_LAUNCH(32, 16) break;
      default: return -2;
    }
  } else {
    return -2;
  }
#undef DELTA_LAUNCH
  return si_last_error();
}

// ---- a decay per key channel -----------------------------------------------------------------------------------------
// dec [T, H * dk] fp32 holds raw values x and receives g = exp(-exp(A_log_h) * softplus(x + dt_bias)) in place; ba: rows with H raw
// values b at b_off in the compute dtype; bg fp32 [T, H + G]: beta = sigmoid(b), then q . k of the (unit) vectors per query/key
// head, which lie in xc as [q: G * dk | k: G * dk | ...]. A warp takes a (row, head) or a (row, query/key head).
template <typename T>
__global__ void __launch_bounds__(256) channel_delta_prepare_kernel(const float* __restrict__ xc, long long xc_stride,
    const T* __restrict__ ba, long long ba_stride, int b_off, float* __restrict__ dec, long long dec_stride,
    const float* __restrict__ a_log, const float* __restrict__ dt_bias, float* __restrict__ bg, long long units, int G, int H, int dk,
    int wide) {
  pdl_prologue();
  const long long unit = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (unit >= units) return;
  const int lane = threadIdx.x & 31;
  const long long t = unit / (H + G);
  const int h = (int)(unit - t * (H + G));
  float* bgr = bg + t * (H + G);
  if (h >= H) {
    const float* q = xc + t * xc_stride + (size_t)(h - H) * dk;
    const float* k = q + (size_t)G * dk;
    float dot = 0.f;
    if (wide) {
      for (int i = lane * 4; i < dk; i += 128) {
        const float4 a = *reinterpret_cast<const float4*>(q + i), b = *reinterpret_cast<const float4*>(k + i);
        dot = fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, dot))));
      }
    } else {
      for (int i = lane; i < dk; i += 32) dot = fmaf(q[i], k[i], dot);
    }
    dot = warp_sum(dot);
    if (lane == 0) bgr[h] = dot;
    return;
  }
  const float rate = expf(a_log[h]);
  float* d = dec + t * dec_stride + (size_t)h * dk;
  const float* bias = dt_bias + (size_t)h * dk;
  auto decay = [&](float x, float b) { return expf(-rate * softplus_d(x + b)); };
  if (wide) {
    for (int i = lane * 4; i < dk; i += 128) {
      const float4 x = *reinterpret_cast<const float4*>(d + i), b = *reinterpret_cast<const float4*>(bias + i);
      *reinterpret_cast<float4*>(d + i) = make_float4(decay(x.x, b.x), decay(x.y, b.y), decay(x.z, b.z), decay(x.w, b.w));
    }
  } else {
    for (int i = lane; i < dk; i += 32) d[i] = decay(d[i], bias[i]);
  }
  if (lane == 0) bgr[h] = 1.f / (1.f + expf(-to_f32<T>(ba[t * ba_stride + b_off + h])));
}

SI_EXPORT int si_channel_delta_prepare(const float* xc, long long xc_stride, const void* ba, int dtype, long long ba_stride, int b_off,
                                       float* dec, long long dec_stride, const float* a_log, const float* dt_bias, float* bg,
                                       int num_tokens, int G, int H, int dk, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (G <= 0 || H <= 0 || dk <= 0) return -2;
  const uintptr_t all = (uintptr_t)xc | (uintptr_t)dec | (uintptr_t)dt_bias;
  const int wide = dk % 4 == 0 && xc_stride % 4 == 0 && dec_stride % 4 == 0 && (all & 15) == 0;
  const long long units = (long long)num_tokens * (H + G);
  const dim3 grid((unsigned)((units + 7) / 8)), block(256);
  if (dtype == SI_BF16)
    si_launch(channel_delta_prepare_kernel<__nv_bfloat16>, grid, block, 0, stream, xc, xc_stride, (const __nv_bfloat16*)ba, ba_stride,
              b_off, dec, dec_stride, a_log, dt_bias, bg, units, G, H, dk, wide);
  else
    si_launch(channel_delta_prepare_kernel<float>, grid, block, 0, stream, xc, xc_stride, (const float*)ba, ba_stride, b_off, dec,
              dec_stride, a_log, dt_bias, bg, units, G, H, dk, wide);
  return si_last_error();
}

// The scan. Shapes and the state's layout as in delta_scan_kernel; a thread keeps its rows of C neighbouring columns, so that what it
// reads of q, k and the decays serves C of them. With C = 2 the four sums of a thread (k . S and q . S of both columns) are added up
// over the NP lanes together, by exchanging halves: the first step leaves a lane the sums of k or those of q, the second one column's, the
// others add that one number; then every lane fetches both columns' u. Shared memory: two buffers of `chunk` tokens of
// [q: RPT * NP | k: RPT * NP | decay: RPT * NP | v: cols | beta, q . k, -, -] (rows beyond dk stay zero).
#define CHANNEL_SLOTS 4
template <int RPT, int NP, int C>
__global__ void __launch_bounds__(256, RPT * C <= 16 ? 2 : 1) channel_delta_scan_kernel(const float* __restrict__ xc, long long xc_stride,
    const float* __restrict__ dec, long long dec_stride, const float* __restrict__ bg, float* __restrict__ state,
    long long state_stride, float* __restrict__ y, long long y_stride, const int* __restrict__ q_start,
    const int* __restrict__ ctx_len, const int* __restrict__ slots, int G, int H, int dk, int dv, int cols, int chunk) {
  extern __shared__ __align__(16) float sm[];
  pdl_prologue();
  const int s = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * cols;
  const int row0 = q_start[s], n = q_start[s + 1] - row0;
  if (n <= 0) return;
  const int pos0 = ctx_len[s] - n;
  const int g = h / (H / G);
  const int p = threadIdx.x % NP, jl = threadIdx.x / NP;
  const int jc = jl * C, j = j0 + jc;                     // the thread's first column, in the block and in the head
  float* S = state + (size_t)slots[s] * state_stride + (size_t)h * RPT * NP * dv + p;
  const size_t s_step = (size_t)dv * NP;
  float2 st[C][RPT / 2];
  bool col_ok[C];
#pragma unroll
  for (int c = 0; c < C; ++c) {
    col_ok[c] = jc + c < cols && j + c < dv;
#pragma unroll
    for (int r = 0; r < RPT / 2; ++r) {
      const float* src = S + (size_t)(2 * r) * s_step + (size_t)(j + c) * NP;
      st[c][r].x = (col_ok[c] && pos0 > 0) ? src[0] : 0.f;
      st[c][r].y = (col_ok[c] && pos0 > 0) ? src[s_step] : 0.f;
    }
  }
  const int dkp = RPT * NP;
  const int per_tok = 3 * dkp + ((cols + 3) & ~3) + 4;
  const int used = min(chunk, n) * per_tok;               // what of a buffer this launch's tokens reach
  for (int idx = threadIdx.x; idx < 2 * used; idx += blockDim.x) sm[idx < used ? idx : chunk * per_tok + idx - used] = 0.f;
  __syncthreads();
  const size_t q_off = (size_t)g * dk, k_off = (size_t)(G + g) * dk, v_off = (size_t)2 * G * dk + (size_t)h * dv + j0, d_off = (size_t)h * dk;
  const int bg_width = H + G;
  const bool wide = dk % 4 == 0 && xc_stride % 4 == 0 && dec_stride % 4 == 0 && (((uintptr_t)xc | (uintptr_t)dec) & 15) == 0;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  // Where rows are aligned and a token is at most 32 * CHANNEL_SLOTS pieces of 16 bytes, every lane knows its pieces once and
  // for all: where they lie in a row of xc or dec and where they go in a token's shared memory.
  const int pr = dk / 4, pieces = 3 * pr + cols / 4;
  const bool quick = wide && cols % 4 == 0 && j0 + cols <= dv && dv % 4 == 0 && pieces <= 32 * CHANNEL_SLOTS;
  int src_off[CHANNEL_SLOTS], dst_off[CHANNEL_SLOTS];     // source of a decay piece: ~offset
#pragma unroll
  for (int q = 0; q < CHANNEL_SLOTS; ++q) {
    const int idx = lane + 32 * q;
    src_off[q] = 0;
    dst_off[q] = -1;
    if (quick && idx < 3 * pr) {
      const int part = idx / pr, i = (idx - part * pr) * 4;
      src_off[q] = part == 2 ? ~(int)(d_off + i) : (int)(part == 0 ? q_off : k_off) + i;
      dst_off[q] = part * dkp + i;
    } else if (quick && idx < pieces) {
      const int e = (idx - 3 * pr) * 4;
      src_off[q] = (int)v_off + e;
      dst_off[q] = 3 * dkp + e;
    }
  }
  auto fetch = [&](int c0, int buf) {                     // a token a warp
    const int cn = min(chunk, n - c0);
    for (int tt = warp; tt < cn; tt += nwarps) {
      float* dst = sm + ((size_t)buf * chunk + tt) * per_tok;
      const size_t t = (size_t)(row0 + c0 + tt);
      const float* row = xc + t * xc_stride;
      const float* drow = dec + t * dec_stride;
      if (quick) {
#pragma unroll
        for (int q = 0; q < CHANNEL_SLOTS; ++q)
          if (dst_off[q] >= 0) delta_cp16(dst + dst_off[q], src_off[q] < 0 ? drow + ~src_off[q] : row + src_off[q]);
      } else {
        const int unit = wide ? 4 : 1;
#pragma unroll
        for (int part = 0; part < 3; ++part) {
          const float* src = part == 0 ? row + q_off : part == 1 ? row + k_off : drow + d_off;
          for (int i = lane * unit; i < dk; i += 32 * unit) {
            if (wide) delta_cp16(dst + part * dkp + i, src + i);
            else delta_cp4(dst + part * dkp + i, src + i);
          }
        }
        for (int e = lane; e < cols; e += 32)
          if (j0 + e < dv) delta_cp4(dst + 3 * dkp + e, row + v_off + e);
      }
      if (lane < 2) delta_cp4(dst + per_tok - 4 + lane, bg + t * bg_width + (lane == 0 ? h : H + g));
    }
    asm volatile("cp.async.commit_group;\n" ::);
  };
  fetch(0, 0);
  int buf = 0;
  for (int c0 = 0; c0 < n; c0 += chunk, buf ^= 1) {
    const int cn = min(chunk, n - c0);
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();                                      // this chunk has arrived, and everyone is done with the other buffer
    if (c0 + chunk < n) fetch(c0 + chunk, buf ^ 1);
    const float* tok = sm + (size_t)buf * chunk * per_tok;
    float* yp = y + (size_t)(row0 + c0) * y_stride + (size_t)h * dv + j;
#pragma unroll 2
    for (int tt = 0; tt < cn; ++tt, tok += per_tok, yp += y_stride) {
      const float4* q4 = reinterpret_cast<const float4*>(tok) + p;
      const float4* k4 = reinterpret_cast<const float4*>(tok + dkp) + p;
      const float4* g4 = reinterpret_cast<const float4*>(tok + 2 * dkp) + p;
      float2 kk[RPT / 2], sk2[C], sq2[C];
#pragma unroll
      for (int c = 0; c < C; ++c) sk2[c] = sq2[c] = make_float2(0.f, 0.f);
#pragma unroll
      for (int i = 0; i < RPT / 4; ++i) {
        const float4 kv = k4[i * NP], qv = q4[i * NP], gv = g4[i * NP];
        kk[2 * i] = make_float2(kv.x, kv.y);
        kk[2 * i + 1] = make_float2(kv.z, kv.w);
#pragma unroll
        for (int c = 0; c < C; ++c) {
          st[c][2 * i] = __fmul2_rn(make_float2(gv.x, gv.y), st[c][2 * i]);
          st[c][2 * i + 1] = __fmul2_rn(make_float2(gv.z, gv.w), st[c][2 * i + 1]);
          sk2[c] = __ffma2_rn(kk[2 * i], st[c][2 * i], sk2[c]);
          sq2[c] = __ffma2_rn(make_float2(qv.x, qv.y), st[c][2 * i], sq2[c]);
          sk2[c] = __ffma2_rn(kk[2 * i + 1], st[c][2 * i + 1], sk2[c]);
          sq2[c] = __ffma2_rn(make_float2(qv.z, qv.w), st[c][2 * i + 1], sq2[c]);
        }
      }
      const float2 sc = *reinterpret_cast<const float2*>(tok + per_tok - 4);      // beta, q . k
      float u[C];
      if constexpr (C == 2) {
        static_assert(NP >= 4, "two columns a thread need four lanes");
        const bool has_q = p & (NP / 2), second = p & (NP / 4);
        const float k0 = sk2[0].x + sk2[0].y, k1 = sk2[1].x + sk2[1].y, q0 = sq2[0].x + sq2[0].y, q1 = sq2[1].x + sq2[1].y;
        const float a0 = (has_q ? q0 : k0) + __shfl_xor_sync(0xffffffffu, has_q ? k0 : q0, NP / 2);
        const float a1 = (has_q ? q1 : k1) + __shfl_xor_sync(0xffffffffu, has_q ? k1 : q1, NP / 2);
        float sum = (second ? a1 : a0) + __shfl_xor_sync(0xffffffffu, second ? a0 : a1, NP / 4);
#pragma unroll
        for (int o = NP / 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        // the lane's column; v beyond the block's columns lies inside the token's padding
        const float mine = sc.x * (tok[3 * dkp + jc + (second ? 1 : 0)] - sum);
        u[0] = __shfl_sync(0xffffffffu, mine, 0, NP);
        u[1] = __shfl_sync(0xffffffffu, mine, NP / 4, NP);
        if ((p == NP / 2 && col_ok[0]) || (p == NP / 2 + NP / 4 && col_ok[1])) yp[second ? 1 : 0] = fmaf(sc.y, second ? u[1] : u[0], sum);
      } else {
        float sk = sk2[0].x + sk2[0].y, sq = sq2[0].x + sq2[0].y;
#pragma unroll
        for (int o = 1; o < NP; o <<= 1) {
          sk += __shfl_xor_sync(0xffffffffu, sk, o);
          sq += __shfl_xor_sync(0xffffffffu, sq, o);
        }
        u[0] = sc.x * (tok[3 * dkp + (col_ok[0] ? jc : 0)] - sk);
        if (p == 0 && col_ok[0]) *yp = fmaf(sc.y, u[0], sq);
      }
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const float2 u2 = make_float2(u[c], u[c]);
#pragma unroll
        for (int r = 0; r < RPT / 2; ++r) st[c][r] = __ffma2_rn(kk[r], u2, st[c][r]);
      }
    }
  }
#pragma unroll
  for (int c = 0; c < C; ++c)
    if (col_ok[c]) {
#pragma unroll
      for (int r = 0; r < RPT / 2; ++r) {
        float* dst = S + (size_t)(2 * r) * s_step + (size_t)(j + c) * NP;
        dst[0] = st[c][r].x;
        dst[s_step] = st[c][r].y;
      }
    }
}

SI_EXPORT int si_channel_delta_scan(const float* xc, long long xc_stride, const float* dec, long long dec_stride, const float* bg,
                                    float* state, long long state_stride, float* y, long long y_stride, const int* q_start,
                                    const int* ctx_len, const int* slots, int num_seqs, int G, int H, int dk, int dv,
                                    cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (G <= 0 || H % G || dk <= 0 || dv <= 0 || dk > 512 || H > 65535) return -2;
  if (2LL * G * dk + (long long)H * dv >= (1LL << 30) || (long long)H * dk >= (1LL << 30)) return -2;
  const DeltaShape sh = delta_shape(dk);
  if (sh.rpt * sh.np < dk || state_stride < (long long)H * sh.rpt * sh.np * dv) return -2;
  const int C = sh.np == 16 ? 2 : 1;                      // columns a thread
  int groups = 256 / sh.np;                               // column groups a block: as in si_delta_scan, a warp at least
  if (groups > (dv + C - 1) / C) groups = (dv + C - 1) / C;
  const long long per = (long long)num_seqs * H;
  while (groups > 1 && (groups / 2) * sh.np >= 32 && per * ((dv + groups * C - 1) / (groups * C)) < si_sm_count()) groups /= 2;
  const int cols = groups * C;
  const int zb = (dv + cols - 1) / cols;
  if (zb > 65535) return -2;
  const int threads = ((groups * sh.np + 31) / 32) * 32;
  const size_t per_tok = (size_t)(3 * sh.np * sh.rpt + ((cols + 3) & ~3) + 4) * sizeof(float);
  int chunk = DELTA_CHUNK;                                // fewer tokens a buffer where two of 32 would not fit
  while (chunk > 1 && 2 * chunk * per_tok > (sh.rpt * C <= 16 ? 110 : 200) * 1024) chunk /= 2;
  const size_t smem = 2 * chunk * per_tok;
  if (smem > 200 * 1024) return -2;
  const dim3 grid(num_seqs, H, zb), block(threads);
#define CHANNEL_LAUNCH(R, P, C)                                                                                       \
  {                                                                                                                  \
    static size_t configured = 0;                                                                                    \
    if (smem > 48 * 1024 && smem > configured) {                                                                     \
      if (cudaFuncSetAttribute(channel_delta_scan_kernel<R, P, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) \
        return -2;                                                                                                   \
      configured = smem;                                                                                             \
    }                                                                                                                \
    si_launch(channel_delta_scan_kernel<R, P, C>, grid, block, smem, stream, xc, xc_stride, dec, dec_stride, bg, state, state_stride, y, \
              y_stride, q_start, ctx_len, slots, G, H, dk, dv, cols, chunk);                                         \
  }
  if (sh.np < 16) {
    if (sh.rpt != 4) return -2;
    switch (sh.np) {
      case 1: CHANNEL_LAUNCH(4, 1, 1) break;
      case 2: CHANNEL_LAUNCH(4, 2, 1) break;
      case 4: CHANNEL_LAUNCH(4, 4, 1) break;
      case 8: CHANNEL_LAUNCH(4, 8, 1) break;
      default: return -2;
    }
  } else if (sh.np == 16) {
    switch (sh.rpt) {
      case 4: CHANNEL_LAUNCH(4, 16, 2) break;
      case 8: CHANNEL_LAUNCH(8, 16, 2) break;
      case 12: CHANNEL_LAUNCH(12, 16, 2) break;
      case 16: CHANNEL_LAUNCH(16, 16, 2) break;
      case 20: CHANNEL_LAUNCH(20, 16, 2) break;
      case 24: CHANNEL_LAUNCH(24, 16, 2) break;
      case 28: CHANNEL_LAUNCH(28, 16, 2) break;
      case 32: CHANNEL_LAUNCH(32, 16, 2) break;
      default: return -2;
    }
  } else {
    return -2;
  }
#undef CHANNEL_LAUNCH
  return si_last_error();
}

// ---- a decay per key channel, four tokens at a time -----------------------------------------------------------------
// For portions of several rows the recurrence runs in groups of four tokens (counted from the portion's start). With c_i the product of
// the group's decays up to token i, s_i that of the decays behind it, C that of all four, S the state before the group, and
//   kk_ij = k_i . diag(g_(j+1) .. g_i) k_j  (j < i),    qk_ij likewise with q_i  (j <= i):
//   u_i = beta_i (v_i - (c_i k_i) . S - sum_(j<i) kk_ij u_j);   o_i = (c_i q_i) . S + sum_(j<=i) qk_ij u_j;   S <- C S + sum_i (s_i k_i) u_i^T
// which is the token-by-token recurrence written out, all in fp32 and with products of decays alone (nothing is divided). The sums over
// the key channels of all four tokens read the same state, so they are formed and added up over the lanes together, and what is left
// of the chain from token to token is a triangular system of a few scalars.
#define GROUP_TOKENS 4
#define GROUP_SCALARS 8                                   // a token's beta, kk_i0 .. kk_i2, qk_i0 .. qk_i3

// rec [T, H, 3, dk]: c_i k_i, c_i q_i, s_i k_i; sc [T, H, 8]; dec [T, H * dk]: raw values, of which the rows that start a group become C.
// A warp takes a (group, head).
// V neighbouring entries that a lane takes at a time (two: with four the sums of a group leave room for fewer warps, 53 against 50 us at
// 16 heads of 128 and 2,048 tokens)
template <int V> struct Piece { float v[V]; };
template <int V> __device__ __forceinline__ Piece<V> piece_load(const float* p) {
  Piece<V> o;
  if constexpr (V == 4) { const float4 t = *reinterpret_cast<const float4*>(p); o.v[0] = t.x; o.v[1] = t.y; o.v[2] = t.z; o.v[3] = t.w; }
  else { const float2 t = *reinterpret_cast<const float2*>(p); o.v[0] = t.x; o.v[1] = t.y; }
  return o;
}
template <int V> __device__ __forceinline__ void piece_store(float* p, const Piece<V>& o) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(o.v[0], o.v[1], o.v[2], o.v[3]);
  else *reinterpret_cast<float2*>(p) = make_float2(o.v[0], o.v[1]);
}

template <typename T>
__global__ void __launch_bounds__(256, 3) channel_delta_groups_kernel(const float* __restrict__ xc, long long xc_stride,
    const T* __restrict__ ba, long long ba_stride, int b_off, float* __restrict__ dec, long long dec_stride,
    const float* __restrict__ a_log, const float* __restrict__ dt_bias, float* __restrict__ rec, float* __restrict__ sc,
    const int* __restrict__ row_seq, const int* __restrict__ q_start, int num_seqs, int G, int H, int dk) {
  pdl_prologue();
  const int t = blockIdx.x, h = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int seq = row_seq[t];
  if (seq < 0 || seq >= num_seqs || h >= H) return;
  if ((t - q_start[seq]) % GROUP_TOKENS) return;
  const int m = min(GROUP_TOKENS, q_start[seq + 1] - t);
  const int gh = h / (H / G);
  const float rate = expf(a_log[h]);
  float dots[16];                                         // qk_00 qk_10 qk_11 qk_20 .. qk_33, kk_10 kk_20 kk_21 kk_30 kk_31 kk_32
#pragma unroll
  for (int v = 0; v < 16; ++v) dots[v] = 0.f;
  constexpr int V = 2;
  for (int i0 = lane * V; i0 < dk; i0 += 32 * V) {
    Piece<V> g[4], k[4], q[4];
    const Piece<V> b = piece_load<V>(dt_bias + (size_t)h * dk + i0);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
#pragma unroll
      for (int e = 0; e < V; ++e) g[i].v[e] = k[i].v[e] = q[i].v[e] = 0.f;
      if (i < m) {
        const float* row = xc + (size_t)(t + i) * xc_stride + (size_t)gh * dk + i0;
        g[i] = piece_load<V>(dec + (size_t)(t + i) * dec_stride + (size_t)h * dk + i0);
        q[i] = piece_load<V>(row);
        k[i] = piece_load<V>(row + (size_t)G * dk);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < V; ++e) g[i].v[e] = i < m ? expf(-rate * softplus_d(g[i].v[e] + b.v[e])) : 1.f;
    Piece<V> c;
#pragma unroll
    for (int e = 0; e < V; ++e) c.v[e] = 1.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      Piece<V> kc, qc, ks;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        c.v[e] *= g[i].v[e];
        kc.v[e] = c.v[e] * k[i].v[e];
        qc.v[e] = c.v[e] * q[i].v[e];
        float w = k[i].v[e];                              // k_i as the tokens behind it in the group see it
        dots[i * (i + 1) / 2 + i] = fmaf(q[i].v[e], w, dots[i * (i + 1) / 2 + i]);
#pragma unroll
        for (int l = i + 1; l < 4; ++l) {
          w *= g[l].v[e];
          dots[l * (l + 1) / 2 + i] = fmaf(q[l].v[e], w, dots[l * (l + 1) / 2 + i]);
          dots[10 + l * (l - 1) / 2 + i] = fmaf(k[l].v[e], w, dots[10 + l * (l - 1) / 2 + i]);
        }
        ks.v[e] = w;
      }
      if (i < m) {
        float* dst = rec + ((size_t)(t + i) * H + h) * 3 * dk + i0;
        piece_store<V>(dst, kc);
        piece_store<V>(dst + dk, qc);
        piece_store<V>(dst + 2 * dk, ks);
      }
    }
    piece_store<V>(dec + (size_t)t * dec_stride + (size_t)h * dk + i0, c);
  }
  // the sixteen sums over the warp by exchanging halves: lanes 2v and 2v + 1 end with sum v
#pragma unroll
  for (int half = 8, bit = 16; half > 0; half >>= 1, bit >>= 1) {
    const bool up = lane & bit;
#pragma unroll
    for (int v = 0; v < half; ++v) {
      const float keep = up ? dots[v + half] : dots[v], send = up ? dots[v] : dots[v + half];
      dots[v] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
    }
  }
  const float dot = dots[0] + __shfl_xor_sync(0xffffffffu, dots[0], 1);
  // where sum v goes (even lanes), and the places that hold no sum (odd lanes, zero): token * 8 + place
  const int v = lane >> 1;
  int i, place;
  if (!(lane & 1)) {
    if (v < 10) { i = v < 1 ? 0 : v < 3 ? 1 : v < 6 ? 2 : 3; place = 4 + v - i * (i + 1) / 2; }
    else { i = v - 10 < 1 ? 1 : v - 10 < 3 ? 2 : 3; place = 1 + v - 10 - i * (i - 1) / 2; }
  } else if (v < 6) {                                     // qk_ij, j > i
    i = v < 3 ? 0 : v < 5 ? 1 : 2; place = 4 + (v < 3 ? 1 + v : v < 5 ? v - 1 : 3);
  } else {                                                // kk_ij, j >= i
    i = v < 9 ? 0 : v < 11 ? 1 : 2; place = 1 + (v < 9 ? v - 6 : v < 11 ? v - 8 : 2);
  }
  if (i < m && !((lane & 1) && v >= 12)) sc[((size_t)(t + i) * H + h) * GROUP_SCALARS + place] = (lane & 1) ? 0.f : dot;
  if (lane < m) sc[((size_t)(t + lane) * H + h) * GROUP_SCALARS] = 1.f / (1.f + expf(-to_f32<T>(ba[(size_t)(t + lane) * ba_stride + b_off + h])));
}

SI_EXPORT int si_channel_delta_groups(const float* xc, long long xc_stride, const void* ba, int dtype, long long ba_stride, int b_off,
                                      float* dec, long long dec_stride, const float* a_log, const float* dt_bias, float* rec, float* sc,
                                      const int* row_seq, const int* q_start, int num_tokens, int num_seqs, int G, int H, int dk,
                                      cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  const uintptr_t all = (uintptr_t)xc | (uintptr_t)dec | (uintptr_t)dt_bias | (uintptr_t)rec;
  if (G <= 0 || H <= 0 || H % G || dk <= 0 || dk % 4 || xc_stride % 4 || dec_stride % 4 || (all & 15)) return -2;
  const dim3 grid(num_tokens, (H + 7) / 8), block(H >= 8 ? 256 : 32 * H);
  if (dtype == SI_BF16)
    si_launch(channel_delta_groups_kernel<__nv_bfloat16>, grid, block, 0, stream, xc, xc_stride, (const __nv_bfloat16*)ba, ba_stride,
              b_off, dec, dec_stride, a_log, dt_bias, rec, sc, row_seq, q_start, num_seqs, G, H, dk);
  else
    si_launch(channel_delta_groups_kernel<float>, grid, block, 0, stream, xc, xc_stride, (const float*)ba, ba_stride, b_off, dec,
              dec_stride, a_log, dt_bias, rec, sc, row_seq, q_start, num_seqs, G, H, dk);
  return si_last_error();
}

// The scan over groups. A thread keeps RPT rows of two neighbouring columns of S, the 16 parts of a column pair are neighbouring lanes
// (shapes and the state's layout as in delta_scan_kernel). A group's sixteen numbers a thread ((c k_i) . S and (c q_i) . S, four tokens, two columns)
// are added up over the 16 lanes by exchanging halves, so that lane p = [q | token | column] ends with one of them; every lane fetches
// the eight that the triangular system needs and solves it for both columns. Shared memory: two buffers of GROUP_AHEAD groups of
// 4 x [c k | c q | s k: RPT * 16 each | v: cols | scalars] and C; every thread knows its pieces of a group once and for all.
#define GROUP_AHEAD 4
template <int RPT, int SLOTS>
__global__ void __launch_bounds__(256, RPT <= 8 && SLOTS <= 4 ? 2 : 1) channel_delta_group_scan_kernel(const float* __restrict__ rec,
    const float* __restrict__ sc, const float* __restrict__ dec, long long dec_stride, const float* __restrict__ xc, long long xc_stride,
    float* __restrict__ state, long long state_stride, float* __restrict__ y, long long y_stride, const int* __restrict__ q_start,
    const int* __restrict__ ctx_len, const int* __restrict__ slots, int G, int H, int dk, int dv, int cols) {
  extern __shared__ __align__(16) float sm[];
  pdl_prologue();
  constexpr int NP = 16, M = GROUP_TOKENS, DKP = RPT * NP;
  const int s = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * cols;
  const int row0 = q_start[s], n = q_start[s + 1] - row0;
  if (n <= 0) return;
  const int pos0 = ctx_len[s] - n, groups = (n + M - 1) / M;
  const int p = threadIdx.x % NP, jc = threadIdx.x / NP * 2, j = j0 + jc;
  const int TOK = 3 * DKP + cols + GROUP_SCALARS, GROUP = M * TOK + DKP;
  float* S = state + (size_t)slots[s] * state_stride + (size_t)h * DKP * dv + p;
  const size_t s_step = (size_t)dv * NP;
  float2 st[2][RPT / 2];
  bool ok[2];
#pragma unroll
  for (int c = 0; c < 2; ++c) {
    ok[c] = j + c < dv;
#pragma unroll
    for (int r = 0; r < RPT / 2; ++r) {
      const float* src = S + (size_t)(2 * r) * s_step + (size_t)(j + c) * NP;
      st[c][r].x = (ok[c] && pos0 > 0) ? src[0] : 0.f;
      st[c][r].y = (ok[c] && pos0 > 0) ? src[s_step] : 0.f;
    }
  }
  for (int idx = threadIdx.x; idx < 2 * GROUP_AHEAD * GROUP; idx += blockDim.x) sm[idx] = 0.f;      // rows beyond dk stay zero
  __syncthreads();
  // this thread's pieces of a group: 4 x [3 dk / 4 of rec | cols / 4 of v | 2 of sc], then dk / 4 of C
  const int pr = 3 * dk / 4, pv = cols / 4, per = pr + pv + 2, pieces = M * per + dk / 4;
  const float* src[SLOTS];
  int dst[SLOTS], tok[SLOTS];                             // place in a group; token of the group (-1: no piece)
  unsigned step[SLOTS];                                   // entries from group to group
#pragma unroll
  for (int q = 0; q < SLOTS; ++q) {
    const int idx = threadIdx.x + q * blockDim.x;
    src[q] = rec; dst[q] = 0; tok[q] = -1; step[q] = 0;
    if (idx < M * per) {
      const int i = idx / per, e = idx - i * per;
      const size_t row = (size_t)(row0 + i);
      tok[q] = i;
      if (e < pr) {
        const int part = e / (dk / 4), at = (e - part * (dk / 4)) * 4;
        src[q] = rec + (row * H + h) * 3 * dk + part * dk + at;
        dst[q] = i * TOK + part * DKP + at;
        step[q] = (unsigned)(M * H * 3 * dk);
      } else if (e < pr + pv) {
        const int at = (e - pr) * 4;
        if (j0 + at >= dv) tok[q] = -1;                   // columns beyond the head's
        src[q] = xc + row * xc_stride + (size_t)2 * G * dk + (size_t)h * dv + j0 + at;
        dst[q] = i * TOK + 3 * DKP + at;
        step[q] = (unsigned)(M * xc_stride);
      } else {
        const int at = (e - pr - pv) * 4;
        src[q] = sc + (row * H + h) * GROUP_SCALARS + at;
        dst[q] = i * TOK + 3 * DKP + cols + at;
        step[q] = (unsigned)(M * H * GROUP_SCALARS);
      }
    } else if (idx < pieces) {
      const int at = (idx - M * per) * 4;
      tok[q] = 0;
      src[q] = dec + (size_t)row0 * dec_stride + (size_t)h * dk + at;
      dst[q] = M * TOK + at;
      step[q] = (unsigned)(M * dec_stride);
    }
  }
  auto fetch = [&](int g0, int buf) {                     // groups in order: the sources move on
    for (int a = 0; a < GROUP_AHEAD; ++a) {
      if (g0 + a >= groups) break;
      float* base = sm + (size_t)(buf * GROUP_AHEAD + a) * GROUP;
      const int left = n - (g0 + a) * M;                  // tokens of the portion from this group on
#pragma unroll
      for (int q = 0; q < SLOTS; ++q) {
        if (tok[q] >= 0) {
          const int bytes = tok[q] < left ? 16 : 0;       // tokens behind the portion are zeros
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"((unsigned)__cvta_generic_to_shared(base + dst[q])),
                       "l"(bytes ? src[q] : rec), "r"(bytes));
          src[q] += step[q];
        }
      }
    }
    asm volatile("cp.async.commit_group;\n" ::);
  };
  fetch(0, 0);
  const bool has_q = p & 8;
  const int my_i = (p >> 1) & 3, my_c = p & 1;
  float* yp = y + (size_t)(row0 + my_i) * y_stride + (size_t)h * dv + j + my_c;
  const bool writes = has_q && j + my_c < dv;
  int buf = 0;
  for (int g0 = 0; g0 < groups; g0 += GROUP_AHEAD, buf ^= 1) {
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();                                      // these groups have arrived, and everyone is done with the other buffer
    if (g0 + GROUP_AHEAD < groups) fetch(g0 + GROUP_AHEAD, buf ^ 1);
    const int ga = min(GROUP_AHEAD, groups - g0);
    for (int a = 0; a < ga; ++a) {
      const float* base = sm + (size_t)(buf * GROUP_AHEAD + a) * GROUP;
      float val[16];                                      // [q | token | column]
#pragma unroll
      for (int i = 0; i < M; ++i) {
        const float4* k4 = reinterpret_cast<const float4*>(base + i * TOK) + p;
        const float4* q4 = reinterpret_cast<const float4*>(base + i * TOK + DKP) + p;
        float2 ak[2], aq[2];
#pragma unroll
        for (int c = 0; c < 2; ++c) ak[c] = aq[c] = make_float2(0.f, 0.f);
#pragma unroll
        for (int r = 0; r < RPT / 4; ++r) {
          const float4 kv = k4[r * NP], qv = q4[r * NP];
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            ak[c] = __ffma2_rn(make_float2(kv.x, kv.y), st[c][2 * r], ak[c]);
            aq[c] = __ffma2_rn(make_float2(qv.x, qv.y), st[c][2 * r], aq[c]);
            ak[c] = __ffma2_rn(make_float2(kv.z, kv.w), st[c][2 * r + 1], ak[c]);
            aq[c] = __ffma2_rn(make_float2(qv.z, qv.w), st[c][2 * r + 1], aq[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          val[2 * i + c] = ak[c].x + ak[c].y;
          val[8 + 2 * i + c] = aq[c].x + aq[c].y;
        }
      }
#pragma unroll
      for (int half = 8; half > 0; half >>= 1) {
        const bool up = p & half;
#pragma unroll
        for (int v = 0; v < half; ++v) {
          const float keep = up ? val[v + half] : val[v], send = up ? val[v] : val[v + half];
          val[v] = keep + __shfl_xor_sync(0xffffffffu, send, half);
        }
      }
      const float mine = val[0];
      float u[M][2];
#pragma unroll
      for (int i = 0; i < M; ++i) {
        const float* t = base + i * TOK + 3 * DKP;
        const float4 bk = *reinterpret_cast<const float4*>(t + cols);      // beta, kk_i0, kk_i1, kk_i2
        const float2 vv = *reinterpret_cast<const float2*>(t + jc);
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          float r = (c ? vv.y : vv.x) - __shfl_sync(0xffffffffu, mine, 2 * i + c, NP);
          if (i > 0) r = fmaf(-bk.y, u[0][c], r);
          if (i > 1) r = fmaf(-bk.z, u[1][c], r);
          if (i > 2) r = fmaf(-bk.w, u[2][c], r);
          u[i][c] = bk.x * r;
        }
      }
      {
        const float4 qk = *reinterpret_cast<const float4*>(base + my_i * TOK + 3 * DKP + cols + 4);      // zeros behind token my_i
        float o = fmaf(qk.x, my_c ? u[0][1] : u[0][0], mine);
        o = fmaf(qk.y, my_c ? u[1][1] : u[1][0], o);
        o = fmaf(qk.z, my_c ? u[2][1] : u[2][0], o);
        o = fmaf(qk.w, my_c ? u[3][1] : u[3][0], o);
        if (writes && (g0 + a) * M + my_i < n) *yp = o;
        yp += M * y_stride;
      }
      const float4* c4 = reinterpret_cast<const float4*>(base + M * TOK) + p;
#pragma unroll
      for (int r = 0; r < RPT / 4; ++r) {
        const float4 cv = c4[r * NP];
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          st[c][2 * r] = __fmul2_rn(make_float2(cv.x, cv.y), st[c][2 * r]);
          st[c][2 * r + 1] = __fmul2_rn(make_float2(cv.z, cv.w), st[c][2 * r + 1]);
        }
#pragma unroll
        for (int i = 0; i < M; ++i) {
          const float4 kv = reinterpret_cast<const float4*>(base + i * TOK + 2 * DKP)[p + r * NP];
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            const float2 u2 = make_float2(u[i][c], u[i][c]);
            st[c][2 * r] = __ffma2_rn(make_float2(kv.x, kv.y), u2, st[c][2 * r]);
            st[c][2 * r + 1] = __ffma2_rn(make_float2(kv.z, kv.w), u2, st[c][2 * r + 1]);
          }
        }
      }
    }
  }
#pragma unroll
  for (int c = 0; c < 2; ++c)
    if (ok[c]) {
#pragma unroll
      for (int r = 0; r < RPT / 2; ++r) {
        float* d = S + (size_t)(2 * r) * s_step + (size_t)(j + c) * NP;
        d[0] = st[c][r].x;
        d[s_step] = st[c][r].y;
      }
    }
}

// 1 when the form by groups takes a state of dk x dv: sixteen parts a column, sizes in multiples of 4.
SI_EXPORT int si_channel_delta_groups_ok(int dk, int dv) {
  if (dk <= 0 || dv <= 0 || dk % 4 || dv % 4 || dk > 256) return 0;
  const DeltaShape sh = delta_shape(dk);
  return sh.np == 16 && sh.rpt <= 16;
}

#define GROUP_COLS 32                                     // most columns a block (16, 64: no faster)
SI_EXPORT int si_channel_delta_group_scan(const float* rec, const float* sc, const float* dec, long long dec_stride, const float* xc,
                                          long long xc_stride, float* state, long long state_stride, float* y, long long y_stride,
                                          const int* q_start, const int* ctx_len, const int* slots, int num_seqs, int G, int H, int dk,
                                          int dv, cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  const uintptr_t all = (uintptr_t)xc | (uintptr_t)dec | (uintptr_t)sc | (uintptr_t)rec;
  if (G <= 0 || H % G || H > 65535 || !si_channel_delta_groups_ok(dk, dv) || xc_stride % 4 || dec_stride % 4 || (all & 15)) return -2;
  if (12LL * H * dk >= (1LL << 31) || 4 * xc_stride >= (1LL << 31)) return -2;
  const DeltaShape sh = delta_shape(dk);
  if (state_stride < (long long)H * sh.rpt * sh.np * dv) return -2;
  // columns a block, a multiple of 4: fewer while the blocks do not fill the device, so that every scheduler has a warp
  int cols = GROUP_COLS;
  while (cols > 8 && cols / 2 >= dv) cols /= 2;
  const long long per = (long long)num_seqs * H;
  while (cols > 16 && per * ((dv + cols - 1) / cols) < si_sm_count()) cols /= 2;
  const int zb = (dv + cols - 1) / cols, threads = cols * 8;
  const int pieces = GROUP_TOKENS * (3 * dk / 4 + cols / 4 + 2) + dk / 4, need = (pieces + threads - 1) / threads;
  const size_t smem = (size_t)2 * GROUP_AHEAD * (GROUP_TOKENS * (3 * sh.rpt * 16 + cols + GROUP_SCALARS) + sh.rpt * 16) * sizeof(float);
  if (zb > 65535 || need > 8 || smem > 220 * 1024) return -2;
  const dim3 grid(num_seqs, H, zb), block(threads);
#define GROUP_LAUNCH(R, Q)                                                                                           \
  {                                                                                                                  \
    static size_t configured = 0;                                                                                    \
    if (smem > 48 * 1024 && smem > configured) {                                                                     \
      if (cudaFuncSetAttribute(channel_delta_group_scan_kernel<R, Q>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) \
        return -2;                                                                                                   \
      configured = smem;                                                                                             \
    }                                                                                                                \
    si_launch(channel_delta_group_scan_kernel<R, Q>, grid, block, smem, stream, rec, sc, dec, dec_stride, xc, xc_stride, state, \
              state_stride, y, y_stride, q_start, ctx_len, slots, G, H, dk, dv, cols);                               \
  }
#define GROUP_LAUNCH_SLOTS(R) { if (need <= 2) GROUP_LAUNCH(R, 2) else if (need <= 4) GROUP_LAUNCH(R, 4) else GROUP_LAUNCH(R, 8) }
  switch (sh.rpt) {
    case 4: GROUP_LAUNCH_SLOTS(4) break;
    case 8: GROUP_LAUNCH_SLOTS(8) break;
    case 12: GROUP_LAUNCH_SLOTS(12) break;
    case 16: GROUP_LAUNCH_SLOTS(16) break;
    default: return -2;
  }
#undef GROUP_LAUNCH_SLOTS
#undef GROUP_LAUNCH
  return si_last_error();
}

// ---- the read-out's norm and gate ------------------------------------------------------------------------------------
//   out[t, h, :] = post * w_h * o[t, h, :] * rsqrt(mean(o[t, h, :]^2) + eps) * gate(z[t, h, :]),   gate silu or sigmoid
// w [dv] shared by the heads (w_head_stride 0) or [H, dv] with one row a head (w_head_stride dv); post one number.
// o fp32, z and out in the compute dtype (z and out views with a row stride). One warp a (row, head).
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* __restrict__ o, long long o_stride, const T* __restrict__ z,
    long long z_stride, const float* __restrict__ w, T* __restrict__ out, long long out_stride, long long pairs, int H, int dv,
    float eps, long long w_head_stride, float post, int sigmoid) {
  pdl_prologue();
  const long long wi = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (wi >= pairs) return;
  const int lane = threadIdx.x & 31;
  const long long t = wi / H;
  const int h = (int)(wi - t * H);
  const float* orow = o + t * o_stride + (size_t)h * dv;
  const T* zr = z + t * z_stride + (size_t)h * dv;
  float ss = 0.f;
  for (int i = lane; i < dv; i += 32) ss += orow[i] * orow[i];
  const float rs = rsqrtf(warp_sum(ss) / (float)dv + eps) * post;
  w += (size_t)h * w_head_stride;
  T* dst = out + t * out_stride + (size_t)h * dv;
  for (int i = lane; i < dv; i += 32) {
    const float zz = to_f32<T>(zr[i]);
    dst[i] = from_f32<T>(orow[i] * rs * w[i] * ((sigmoid ? 1.f : zz) / (1.f + expf(-zz))));
  }
}

SI_EXPORT int si_head_norm_gate(const float* o, long long o_stride, const void* z, int dtype, long long z_stride,
                                const float* w, void* out, long long out_stride, int rows, int H, int dv, float eps,
                                long long w_head_stride, float post, int sigmoid, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || dv <= 0) return -2;
  const long long pairs = (long long)rows * H;
  const dim3 grid((unsigned)((pairs + 7) / 8)), block(256);
  if (dtype == SI_BF16)
    si_launch(head_norm_gate_kernel<__nv_bfloat16>, grid, block, 0, stream, o, o_stride, (const __nv_bfloat16*)z, z_stride, w,
              (__nv_bfloat16*)out, out_stride, pairs, H, dv, eps, w_head_stride, post, sigmoid);
  else
    si_launch(head_norm_gate_kernel<float>, grid, block, 0, stream, o, o_stride, (const float*)z, z_stride, w, (float*)out,
              out_stride, pairs, H, dv, eps, w_head_stride, post, sigmoid);
  return si_last_error();
}
