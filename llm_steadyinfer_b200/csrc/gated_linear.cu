// The real-gated linear recurrence: every channel is a recurrence of its own with a decay and an input gate made of the input,
//   r = sigmoid(zr + br);   i = sigmoid(zi + bi);   log a = -c r softplus(lam);   a = exp(log a)
//   S_t = a S_(t-1) + sqrt(1 - a^2) i u_t;          out_t = scale * S_t * gelu_tanh(y_t + by)
// zr and zi are block-diagonal products of u (made before this launch, fp32); everything here is fp32. S starts at zero, and a
// portion of a sequence goes on from what the request's slot holds.
//
// Portions: a block takes (sequence, 16 channels) and walks the rows in rounds of 32 segments x 8 rows. A thread (channel,
// segment) makes a and the input of its eight rows, folds them into one pair (A, B) with S -> A S + B, gets the state before its
// segment from the pairs of the segments before it (in shared memory, in order), and walks its rows again from registers. Half a
// warp reads 16 neighbouring channels of a row.
// Sequences of one row (decode): a thread a channel.
#include "common.cuh"
#include <math.h>

#define LRU_CH 16
#define LRU_SEG 32
#define LRU_RP 8

struct LruArgs {
  const float* u; long long u_stride;                    // [T, W] fp32
  const float* z; int bs; long long z_block;             // row (b, t) of the gates at z + b * z_block + t * 2 bs: [r: bs | i: bs]
  const float* br; const float* bi; const float* sp;     // [W]: biases, c * softplus(lam)
  const void* y; long long y_stride; const float* by;    // the other branch's product [T, W], its bias [W] (may be null)
  float* state; long long state_stride;
  void* out; long long out_stride; float scale;
  const int* q_start; const int* ctx_len; const int* slots;
  int W;
};

struct LruRow { float a, b; };
__device__ __forceinline__ float lru_sigmoid(float x) { return __fdividef(1.f, 1.f + expf(-x)); }      // (1 + e^-x beyond 2^126: 0)
// gelu_tanh: 0.5 v (1 + tanh(w)) = v sigmoid(2 w)
__device__ __forceinline__ float lru_gelu(float v) { return v * lru_sigmoid(1.5957691216057308f * (v + 0.044715f * v * v * v)); }

__device__ __forceinline__ LruRow lru_row(float zr, float zi, float u, float sp) {
  const float e = expm1f(-sp * lru_sigmoid(zr));          // a - 1, so that 1 - a^2 = -e (2 + e) keeps its digits near a = 1
  float root;
  asm("sqrt.approx.f32 %0, %1;" : "=f"(root) : "f"(-e * (2.f + e)));
  LruRow o;
  o.a = 1.f + e;
  o.b = root * lru_sigmoid(zi) * u;
  return o;
}

template <typename T>
__global__ void __launch_bounds__(LRU_CH * LRU_SEG, 1) lru_portion_kernel(const LruArgs p) {
  __shared__ float2 fold[LRU_SEG][LRU_CH];
  __shared__ float last[LRU_CH];
  pdl_prologue();
  const int s = blockIdx.y, row0 = p.q_start[s], n = p.q_start[s + 1] - row0;
  if (n <= 1) return;                                    // a single row is the other kernel's
  const int pos0 = p.ctx_len[s] - n;
  const int ch = threadIdx.x % LRU_CH, seg = threadIdx.x / LRU_CH, c = blockIdx.x * LRU_CH + ch;
  const bool on = c < p.W;
  const int cc = on ? c : 0, blk = cc / p.bs, j = cc % p.bs;
  float* slot = p.state + (size_t)p.slots[s] * p.state_stride + cc;
  float S0 = on && pos0 > 0 ? *slot : 0.f;               // the state before the round
  const float br = p.br[cc], bi = p.bi[cc], sp = p.sp[cc], by = p.by ? p.by[cc] : 0.f;
  const float* z = p.z + blk * p.z_block + j;
  const int mine = seg * LRU_RP;                         // the segment's first row in a round
  float zr[LRU_RP], zi[LRU_RP], u[LRU_RP], y[LRU_RP];
  auto load = [&](int c0) {
#pragma unroll
    for (int r = 0; r < LRU_RP; ++r) {
      const int t = c0 + mine + r;
      zr[r] = zi[r] = u[r] = y[r] = 0.f;
      if (t < n) {
        const size_t row = (size_t)(row0 + t);
        zr[r] = z[row * 2 * p.bs];
        zi[r] = z[row * 2 * p.bs + p.bs];
        u[r] = p.u[row * p.u_stride + cc];
        y[r] = to_f32<T>(((const T*)p.y)[row * p.y_stride + cc]);
      }
    }
  };
  load(0);
  for (int c0 = 0; c0 < n; c0 += LRU_SEG * LRU_RP) {
    float a[LRU_RP], b[LRU_RP], yg[LRU_RP];
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int r = 0; r < LRU_RP; ++r) {
      const LruRow o = lru_row(zr[r] + br, zi[r] + bi, u[r], sp);
      const bool have = c0 + mine + r < n;               // rows behind the portion leave the state as it is
      a[r] = have ? o.a : 1.f;
      b[r] = have ? o.b : 0.f;
      A *= a[r];
      B = fmaf(a[r], B, b[r]);
      yg[r] = y[r];
    }
    if (c0 + LRU_SEG * LRU_RP < n) load(c0 + LRU_SEG * LRU_RP);      // the next round's rows are on their way meanwhile
    fold[seg][ch] = make_float2(A, B);
    __syncthreads();
    float S = S0;
#pragma unroll 4
    for (int k = 0; k < seg; ++k) { const float2 f = fold[k][ch]; S = fmaf(f.x, S, f.y); }
#pragma unroll
    for (int r = 0; r < LRU_RP; ++r) {
      const int t = c0 + mine + r;
      S = fmaf(a[r], S, b[r]);
      if (on && t < n) ((T*)p.out)[(size_t)(row0 + t) * p.out_stride + c] = from_f32<T>(p.scale * S * lru_gelu(yg[r] + by));
    }
    if (seg == LRU_SEG - 1) last[ch] = S;
    __syncthreads();                                     // everyone has read the pairs, and the round's last state is there
    S0 = last[ch];
  }
  if (on && seg == 0) *slot = S0;
}

template <typename T>
__global__ void __launch_bounds__(128) lru_row_kernel(const LruArgs p, int trigger) {
  if (trigger) pdl_trigger();
  const int s = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int row = p.q_start[s], n = p.q_start[s + 1] - row;
  const int pos0 = p.ctx_len[s] - n;
  pdl_wait();
  if (n != 1 || c >= p.W) return;
  const int blk = c / p.bs, j = c % p.bs;
  float* slot = p.state + (size_t)p.slots[s] * p.state_stride + c;
  const float* z = p.z + blk * p.z_block + (size_t)row * 2 * p.bs + j;
  const LruRow o = lru_row(z[0] + p.br[c], z[p.bs] + p.bi[c], p.u[(size_t)row * p.u_stride + c], p.sp[c]);
  const float S = fmaf(o.a, pos0 > 0 ? *slot : 0.f, o.b);
  *slot = S;
  const float y = to_f32<T>(((const T*)p.y)[(size_t)row * p.y_stride + c]) + (p.by ? p.by[c] : 0.f);
  ((T*)p.out)[(size_t)row * p.out_stride + c] = from_f32<T>(p.scale * S * lru_gelu(y));
}

// `kinds`: what the step holds, 1 sequences of one row, 2 longer portions, 3 both. `launches` (may be null): kernels launched.
SI_EXPORT int si_gated_linear(const float* u, long long u_stride, const float* z, int bs, long long z_block, const float* br,
                              const float* bi, const float* sp, const void* y, int dtype, long long y_stride, const float* by,
                              float* state, long long state_stride, void* out, long long out_stride, float scale,
                              const int* q_start, const int* ctx_len, const int* slots, int num_seqs, int W, int kinds,
                              int* launches, cudaStream_t stream) {
  if (launches) *launches = 0;
  if (num_seqs <= 0) return 0;
  if (W <= 0 || bs <= 0 || W % bs || num_seqs > 65535 || state_stride < W) return -2;
  const LruArgs p{u, u_stride, z, bs, z_block, br, bi, sp, y, y_stride, by, state, state_stride, out, out_stride, scale,
                  q_start, ctx_len, slots, W};
  int count = 0;
  if (kinds & 2) {
    const dim3 grid((W + LRU_CH - 1) / LRU_CH, num_seqs), block(LRU_CH * LRU_SEG);
    if (dtype == SI_BF16) si_launch(lru_portion_kernel<__nv_bfloat16>, grid, block, 0, stream, p);
    else si_launch(lru_portion_kernel<float>, grid, block, 0, stream, p);
    ++count;
  }
  if (kinds & 1) {
    const dim3 grid((W + 127) / 128, num_seqs);
    const int trigger = si_pdl_trigger_mode((long long)grid.x * grid.y, 8LL * si_sm_count()) == 1;
    if (dtype == SI_BF16) si_launch(lru_row_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, p, trigger);
    else si_launch(lru_row_kernel<float>, grid, dim3(128), 0, stream, p, trigger);
    ++count;
  }
  if (launches) *launches = count;
  return si_last_error();
}
