// The add into the residual stream where the norms around it are of different kinds:
//   d = delta (+ delta_bias);   d' = the delta's own norm of d;   h = resid + d';   resid <- h (not with `rows`)
//   out = the stream's norm of h
// Kinds of a norm:  0 copy    y = x
//                   1 tanh    y = tanh(alpha x) * w + b           entry by entry, no statistics of the row
//                   2 rms     y = w * x * rsqrt(mean(x^2) + eps)
// so that a sublayer's result passes the norm behind it, joins the stream and the stream passes the norm before the next
// sublayer in one launch, whatever the kinds; `out` with kind 0 is the stream itself in the compute dtype. The stream, the
// norms and all sums are fp32. With `rows` output row r comes from stream row rows[r] and the stream stays as it is.
//
// Without a row statistic nothing ties a row's entries together, and the blocks share a row where rows are few; with one a
// block takes a row. Widths that are multiples of 8 (16-byte aligned tensors): eight entries a thread and load, the row in
// registers from the first load to the last store. Other widths: a plain loop.
#include "common.cuh"

enum : int { NORM_COPY = 0, NORM_TANH = 1, NORM_RMS = 2 };

struct KindNorm {
  int kind;
  const float* w; const float* b;                // tanh: weight and bias; rms: weight
  float alpha;                                   // tanh: factor of the argument; rms: eps
};

struct StreamAdd {
  float* resid; const void* delta; const float* delta_bias; const int* rows; void* out;
  KindNorm dn, on;
  int hidden, trigger;
};

template <typename T> __device__ __forceinline__ void ld8(const T* p, float (&v)[8]);
template <> __device__ __forceinline__ void ld8<float>(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <> __device__ __forceinline__ void ld8<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(h[i]);
    v[2 * i] = f.x; v[2 * i + 1] = f.y;
  }
}
template <typename T> __device__ __forceinline__ void st8(T* p, const float (&v)[8]);
template <> __device__ __forceinline__ void st8<float>(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
template <> __device__ __forceinline__ void st8<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 raw;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = raw;
}

// y = the norm of x for eight neighbouring entries from `i` on; inv: the row's rsqrt for the rms kind
__device__ __forceinline__ void apply8(const KindNorm& n, int i, float inv, float (&x)[8]) {
  if (n.kind == NORM_COPY) return;
  float w[8];
  ld8<float>(n.w + i, w);
  if (n.kind == NORM_TANH) {
    float b[8];
    ld8<float>(n.b + i, b);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] = fmaf(tanhf(n.alpha * x[e]), w[e], b[e]);
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] = w[e] * (x[e] * inv);
  }
}
__device__ __forceinline__ float apply1(const KindNorm& n, int i, float inv, float x) {
  if (n.kind == NORM_TANH) return fmaf(tanhf(n.alpha * x), n.w[i], n.b[i]);
  if (n.kind == NORM_RMS) return n.w[i] * (x * inv);
  return x;
}

// CHUNKS: pieces of eight entries a thread; blockIdx.y: the row's share (1 share where a norm has a row statistic)
template <typename T, int CHUNKS>
__global__ void __launch_bounds__(512) stream_add_vec_kernel(const StreamAdd p) {
  __shared__ float scratch[33];
  if (p.trigger) pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x, src = p.rows ? p.rows[r] : r;
  float* h = p.resid + (size_t)src * p.hidden;
  const int nchunks = p.hidden >> 3, first = blockIdx.y * blockDim.x + threadIdx.x, step = blockDim.x * gridDim.y;
  float x[CHUNKS][8], d[CHUNKS][8];
#pragma unroll
  for (int c = 0; c < CHUNKS; ++c) {
    const int i = first + c * step;
    if (i < nchunks) {
      ld8<float>(h + i * 8, x[c]);
      if (p.delta) ld8<T>((const T*)p.delta + (size_t)src * p.hidden + i * 8, d[c]);
    }
  }
  float inv = 1.f;
  if (p.delta) {
    if (p.delta_bias) {
#pragma unroll
      for (int c = 0; c < CHUNKS; ++c) {
        const int i = first + c * step;
        if (i < nchunks) {
          float b[8];
          ld8<float>(p.delta_bias + i * 8, b);
#pragma unroll
          for (int e = 0; e < 8; ++e) d[c][e] += b[e];
        }
      }
    }
    if (p.dn.kind == NORM_RMS) {
      float ss = 0.f;
#pragma unroll
      for (int c = 0; c < CHUNKS; ++c)
        if (first + c * step < nchunks) {
#pragma unroll
          for (int e = 0; e < 8; ++e) ss = fmaf(d[c][e], d[c][e], ss);
        }
      inv = rsqrtf(block_sum(ss, scratch) / (float)p.hidden + p.dn.alpha);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < CHUNKS; ++c) {
    const int i = first + c * step;
    if (i < nchunks && p.delta) {
      apply8(p.dn, i * 8, inv, d[c]);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[c][e] += d[c][e];
      if (!p.rows) st8<float>(h + i * 8, x[c]);
    }
    if (i < nchunks && p.on.kind == NORM_RMS) {
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(x[c][e], x[c][e], ss);
    }
  }
  if (!p.out) return;
  if (p.on.kind == NORM_RMS) inv = rsqrtf(block_sum(ss, scratch) / (float)p.hidden + p.on.alpha);
#pragma unroll
  for (int c = 0; c < CHUNKS; ++c) {
    const int i = first + c * step;
    if (i < nchunks) {
      apply8(p.on, i * 8, inv, x[c]);
      st8<T>((T*)p.out + (size_t)r * p.hidden + i * 8, x[c]);
    }
  }
}

// Any width: a block a row, what is not kept is formed again.
template <typename T>
__global__ void __launch_bounds__(256) stream_add_kernel(const StreamAdd p) {
  __shared__ float scratch[33];
  pdl_prologue();
  const int r = blockIdx.x, src = p.rows ? p.rows[r] : r;
  float* h = p.resid + (size_t)src * p.hidden;
  const T* dl = p.delta ? (const T*)p.delta + (size_t)src * p.hidden : nullptr;
  auto raw = [&](int i) { return to_f32<T>(dl[i]) + (p.delta_bias ? p.delta_bias[i] : 0.f); };
  float dinv = 1.f, inv = 1.f;
  if (dl && p.dn.kind == NORM_RMS) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) { const float v = raw(i); ss = fmaf(v, v, ss); }
    dinv = rsqrtf(block_sum(ss, scratch) / (float)p.hidden + p.dn.alpha);
  }
  const bool stored = dl && !p.rows;             // the sum lies in the stream for the second pass
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
    float v = h[i];
    if (dl) v += apply1(p.dn, i, dinv, raw(i));
    if (stored) h[i] = v;
    ss = fmaf(v, v, ss);
    if (p.out && p.on.kind != NORM_RMS) ((T*)p.out)[(size_t)r * p.hidden + i] = from_f32<T>(apply1(p.on, i, 1.f, v));
  }
  if (!p.out || p.on.kind != NORM_RMS) return;
  inv = rsqrtf(block_sum(ss, scratch) / (float)p.hidden + p.on.alpha);
  for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
    float v = h[i];
    if (dl && !stored) v += apply1(p.dn, i, dinv, raw(i));
    ((T*)p.out)[(size_t)r * p.hidden + i] = from_f32<T>(apply1(p.on, i, inv, v));
  }
}

template <typename T>
static int stream_add_launch(StreamAdd p, int num_rows, cudaStream_t stream) {
  const auto al = [](const void* q) { return ((uintptr_t)q % 16) == 0; };
  const int nchunks = p.hidden / 8;
  if (p.hidden % 8 == 0 && nchunks <= 4 * 512 && al(p.resid) && al(p.delta) && al(p.delta_bias) && al(p.out) && al(p.dn.w) && al(p.dn.b) &&
      al(p.on.w) && al(p.on.b)) {
    const bool rowwise = (p.delta && p.dn.kind == NORM_RMS) || (p.out && p.on.kind == NORM_RMS);
    int threads = nchunks > 256 ? 512 : (nchunks > 128 ? 256 : 128), shares = 1;
    if (!rowwise) {
      threads = nchunks >= 256 ? 256 : 128;
      if (num_rows < 1024) threads = 128;
      shares = si_row_shares(num_rows, nchunks, threads);
    } else if (num_rows >= 1024 && nchunks <= 1024) {
      threads = threads < 256 ? threads : 256;   // many rows: more blocks a multiprocessor
    }
    while (nchunks > 4 * threads * shares) { if (threads < 512) threads *= 2; else ++shares; }
    const int per = (nchunks + threads * shares - 1) / (threads * shares);
    p.trigger = si_pdl_trigger_enabled() && (long long)num_rows * shares <= 2LL * si_sm_count();
    const dim3 grid(num_rows, shares);
    if (per <= 1) si_launch(stream_add_vec_kernel<T, 1>, grid, dim3(threads), 0, stream, p);
    else if (per <= 2) si_launch(stream_add_vec_kernel<T, 2>, grid, dim3(threads), 0, stream, p);
    else si_launch(stream_add_vec_kernel<T, 4>, grid, dim3(threads), 0, stream, p);
    return si_last_error();
  }
  si_launch(stream_add_kernel<T>, dim3(num_rows), dim3(p.hidden >= 1024 ? 256 : 128), 0, stream, p);
  return si_last_error();
}

// dtype: of delta and out. Returns 0, a CUDA error code, or -2 (refused).
SI_EXPORT int si_stream_add(float* resid, const void* delta, const float* delta_bias, int delta_kind, const float* delta_w,
                            const float* delta_b, float delta_alpha, const int* rows, void* out, int out_kind, const float* out_w,
                            const float* out_b, float out_alpha, int dtype, int num_rows, int hidden, cudaStream_t stream) {
  if (num_rows <= 0 || hidden <= 0) return 0;
  const auto bad = [](int kind, const float* w, const float* b) {
    return kind < NORM_COPY || kind > NORM_RMS || (kind != NORM_COPY && !w) || (kind == NORM_TANH && !b);
  };
  if ((delta && bad(delta_kind, delta_w, delta_b)) || (out && bad(out_kind, out_w, out_b)) || (rows && !out)) return -2;
  StreamAdd p{resid, delta, delta_bias, rows, out, KindNorm{delta_kind, delta_w, delta_b, delta_alpha},
              KindNorm{out_kind, out_w, out_b, out_alpha}, hidden, 0};
  return dtype == SI_BF16 ? stream_add_launch<__nv_bfloat16>(p, num_rows, stream) : stream_add_launch<float>(p, num_rows, stream);
}
