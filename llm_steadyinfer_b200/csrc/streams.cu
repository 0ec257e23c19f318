// A residual stream in several copies ("streams", learned connections between them) and the norm of what a sublayer reads:
//   x'_t = sum_s mix[s, t] x_s + write[t] * y        for every stream t, from the old x_s    (without y: x' = x)
//   u    = sum_s read[s] x'_s                         (read absent: the plain sum)
//   out  = weight * u * rsqrt(mean(u^2) + eps)
// One launch between two sublayers: y is the result of the sublayer before, mix and write its connections, read those
// of the sublayer after. Everything is fp32 but y and out (compute dtype); the rows of x are [S, width].
//   * Before the first sublayer all streams are the same row: `src` then holds one row a token (stream stride 0), so
//     the copies are never written out before they differ.
//   * With `rows` the launch reads stream rows rows[r] and stores none (the rows whose logits are wanted).
//   * Few rows (decode): a cluster of up to 8 blocks shares a row, each takes a part of the width, and the blocks add their
//     parts of the sum of squares over distributed shared memory; blocks behind the rows fetch the next product's weights
//     into L2 ahead (a hint).
// The row's new streams are formed in registers: every thread holds its columns of all streams, all loads of a row in
// flight before the first use. Widths and stream counts outside that take the plain kernel at the end.
#include "common.cuh"
#include <cooperative_groups.h>

struct StreamArgs {
  const float* src; long long src_row, src_stream;      // strides in elements; src_stream 0: one row for all streams
  float* dst;                                            // [rows, S, width] or nullptr: nothing is stored
  const void* y;                                         // [rows, width] or nullptr: the streams stay as they are
  const float* mix;                                      // [S, S], [from, to]
  const float* write;                                    // [S]
  const float* read;                                     // [S] or nullptr: ones
  const int* rows;
  const void* weight; int weight_bf16;
  void* out;
  int S, width, num_rows;
  float eps;
  const void* ahead; long long ahead_bytes;
  int trigger;
};

template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T> __device__ __forceinline__ void store4(T* p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = raw;
}
__device__ __forceinline__ void axpy4(float4& a, float f, const float4& x) {
  a.x = fmaf(f, x.x, a.x); a.y = fmaf(f, x.y, a.y); a.z = fmaf(f, x.z, a.z); a.w = fmaf(f, x.w, a.w);
}

// SM streams at most (exactly SM when EXACT); V pieces of four columns a thread.
template <typename T, int SM, bool EXACT, int V>
__global__ void __launch_bounds__(512) stream_norm_vec_kernel(const StreamArgs p) {
  namespace cg = cooperative_groups;
  __shared__ float scratch[33];
  __shared__ float coef[SM * SM + 2 * SM];               // mix, write, read
  __shared__ float part;
  cg::cluster_group cluster = cg::this_cluster();
  const int parts = (int)cluster.num_blocks(), rank = (int)cluster.block_rank();
  const int S = EXACT ? SM : p.S;
  if (p.trigger) pdl_trigger();
  const int r = blockIdx.x / parts;
  if (r >= p.num_rows) {                                 // blocks behind the rows (whole clusters) only fetch ahead
    l2_prefetch_share(p.ahead, p.ahead_bytes, blockIdx.x - p.num_rows * parts, gridDim.x - p.num_rows * parts);
    return;
  }
  const bool moved = p.y != nullptr;
  for (int i = threadIdx.x; i < SM * SM; i += blockDim.x)
    coef[i] = (moved && i / SM < S && i % SM < S) ? p.mix[(i / SM) * S + i % SM] : 0.f;
  for (int i = threadIdx.x; i < SM; i += blockDim.x) {
    coef[SM * SM + i] = (moved && i < S) ? p.write[i] : 0.f;
    coef[SM * SM + SM + i] = i < S ? (p.read ? p.read[i] : 1.f) : 0.f;
  }
  pdl_wait();
  const int row = p.rows ? p.rows[r] : r;
  const int pieces = p.width / 4, per = (pieces + parts - 1) / parts;
  const int c0 = rank * per, c1 = min(pieces, c0 + per);
  const float* src = p.src + (size_t)row * p.src_row;
  const T* y = (const T*)p.y + (size_t)row * p.width;
  float4 x[V][SM], yv[V];
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int c = c0 + threadIdx.x + v * blockDim.x;
    if (c < c1) {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (EXACT || s < S) x[v][s] = load4<float>(src + (size_t)s * p.src_stream + 4 * c);
      if (moved) yv[v] = load4<T>(y + 4 * c);
    }
  }
  __syncthreads();                                       // the coefficients stand
  float4 u[V];
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int c = c0 + threadIdx.x + v * blockDim.x;
    u[v] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < c1) {
      if (moved) {
#pragma unroll
        for (int t = 0; t < SM; ++t) {
          if (!EXACT && t >= S) break;
          float4 n = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
          for (int s = 0; s < SM; ++s)
            if (EXACT || s < S) axpy4(n, coef[s * SM + t], x[v][s]);
          axpy4(n, coef[SM * SM + t], yv[v]);
          axpy4(u[v], coef[SM * SM + SM + t], n);
          if (p.dst) store4<float>(p.dst + ((size_t)r * S + t) * p.width + 4 * c, n);
        }
      } else {
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (EXACT || s < S) axpy4(u[v], coef[SM * SM + SM + s], x[v][s]);
      }
      ss = fmaf(u[v].x, u[v].x, fmaf(u[v].y, u[v].y, fmaf(u[v].z, u[v].z, fmaf(u[v].w, u[v].w, ss))));
    }
  }
  ss = block_sum(ss, scratch);
  if (parts > 1) {                                       // the row's other parts, in the order of the blocks
    if (threadIdx.x == 0) part = ss;
    cluster.sync();
    ss = 0.f;
    for (int b = 0; b < parts; ++b) ss += *cluster.map_shared_rank(&part, b);
    cluster.barrier_arrive();                            // this block has read the others' parts
  }
  const float inv = rsqrtf(ss / (float)p.width + p.eps);
  T* out = (T*)p.out + (size_t)r * p.width;
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int c = c0 + threadIdx.x + v * blockDim.x;
    if (c < c1) {
      const float4 w = p.weight_bf16 ? load4<__nv_bfloat16>((const __nv_bfloat16*)p.weight + 4 * c)
                                     : load4<float>((const float*)p.weight + 4 * c);
      store4<T>(out + 4 * c, make_float4(w.x * (u[v].x * inv), w.y * (u[v].y * inv), w.z * (u[v].z * inv), w.w * (u[v].w * inv)));
    }
  }
  if (parts > 1) cluster.barrier_wait();                 // no block leaves while another may still read its part
}

// Any width and any number of streams: a column at a time, the column's streams and the row of u in shared memory.
template <typename T>
__global__ void stream_norm_kernel(const StreamArgs p) {
  extern __shared__ float sm[];                          // u [width], then [S][threads]
  __shared__ float scratch[33];
  pdl_prologue();
  const int r = blockIdx.x;
  const int row = p.rows ? p.rows[r] : r;
  const int S = p.S;
  float* u = sm;
  float* x = sm + p.width + threadIdx.x;                 // stream s at x[s * blockDim.x]
  const float* src = p.src + (size_t)row * p.src_row;
  const T* y = (const T*)p.y + (size_t)row * p.width;
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
    for (int s = 0; s < S; ++s) x[s * blockDim.x] = src[(size_t)s * p.src_stream + c];
    float acc = 0.f;
    if (p.y) {
      const float yc = to_f32<T>(y[c]);
      for (int t = 0; t < S; ++t) {
        float n = 0.f;
        for (int s = 0; s < S; ++s) n = fmaf(p.mix[s * S + t], x[s * blockDim.x], n);
        n = fmaf(p.write[t], yc, n);
        acc = fmaf(p.read ? p.read[t] : 1.f, n, acc);
        if (p.dst) p.dst[((size_t)r * S + t) * p.width + c] = n;
      }
    } else {
      for (int s = 0; s < S; ++s) acc = fmaf(p.read ? p.read[s] : 1.f, x[s * blockDim.x], acc);
    }
    u[c] = acc;
    ss = fmaf(acc, acc, ss);
  }
  ss = block_sum(ss, scratch);
  const float inv = rsqrtf(ss / (float)p.width + p.eps);
  T* out = (T*)p.out + (size_t)r * p.width;
  for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
    const float w = p.weight_bf16 ? __bfloat162float(((const __nv_bfloat16*)p.weight)[c]) : ((const float*)p.weight)[c];
    out[c] = from_f32<T>(w * (u[c] * inv));
  }
}

// ---- host side --------------------------------------------------------------------------------------------
template <typename T, int SM, bool EXACT, int V>
static int stream_launch_vec(const StreamArgs& p, int blocks, int threads, int parts, cudaStream_t stream) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(blocks);
  cfg.blockDim = dim3(threads);
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (parts > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = parts; attr[n].val.clusterDim.y = 1; attr[n].val.clusterDim.z = 1;
    ++n;
  }
  if (si_pdl_enabled()) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
  }
  cfg.attrs = attr;
  cfg.numAttrs = n;
  cudaLaunchKernelEx(&cfg, stream_norm_vec_kernel<T, SM, EXACT, V>, p);
  return si_last_error();
}

template <typename T, int SM, bool EXACT>
static int stream_launch_pieces(const StreamArgs& p, int blocks, int threads, int parts, int v, cudaStream_t stream) {
  if (v <= 1) return stream_launch_vec<T, SM, EXACT, 1>(p, blocks, threads, parts, stream);
  if constexpr (SM <= 4) {
    if (v > 2) return stream_launch_vec<T, SM, EXACT, 4>(p, blocks, threads, parts, stream);
  }
  return stream_launch_vec<T, SM, EXACT, 2>(p, blocks, threads, parts, stream);
}

template <typename T>
static int stream_launch(StreamArgs p, cudaStream_t stream) {
  const auto al = [](const void* q, unsigned a) { return ((uintptr_t)q % a) == 0; };
  const int pieces = p.width / 4, max_v = p.S > 4 ? 2 : 4, sms = si_sm_count();
  bool vec = p.S <= 8 && p.width % 4 == 0 && p.src_row % 4 == 0 && p.src_stream % 4 == 0 && al(p.src, 16) && al(p.dst, 16) &&
             al(p.y, 4 * sizeof(T)) && al(p.out, 4 * sizeof(T)) && al(p.weight, p.weight_bf16 ? 8 : 16);
  // Blocks that share a row of 2,048 columns or more, while the rows alone leave most of the device idle (measured: shorter
  // rows are done sooner by one block than the cluster's two barriers take)
  int parts = 1;
  while (pieces >= 512 && parts < 8 && (long long)p.num_rows * parts * 2 <= sms && pieces / (parts * 2) >= 64) parts *= 2;
  int per = (pieces + parts - 1) / parts;
  while (parts < 8 && per > max_v * 512) { parts *= 2; per = (pieces + parts - 1) / parts; }
  if (per > max_v * 512) vec = false;
  if (vec) {
    // one piece a thread while that is at most 256 threads (few rows), else as many pieces as keep a block at 256
    int threads = 128;
    while (threads < 256 && per > threads) threads *= 2;
    if (per > max_v * threads) threads = 512;
    const int v = (per + threads - 1) / threads;
    if (p.ahead && p.ahead_bytes < 4096) p.ahead = nullptr;
    p.trigger = si_pdl_trigger_enabled() && (long long)p.num_rows * parts <= sms;       // a launch of one wave
    int extra = 0;
    if (p.ahead) extra = ((sms > p.num_rows * parts ? sms - p.num_rows * parts : 0) + sms) / parts * parts;
    const int blocks = p.num_rows * parts + extra;
    switch (p.S) {
      case 1: return stream_launch_pieces<T, 1, true>(p, blocks, threads, parts, v, stream);
      case 2: return stream_launch_pieces<T, 2, true>(p, blocks, threads, parts, v, stream);
      case 3: return stream_launch_pieces<T, 3, true>(p, blocks, threads, parts, v, stream);
      case 4: return stream_launch_pieces<T, 4, true>(p, blocks, threads, parts, v, stream);
      default: return stream_launch_pieces<T, 8, false>(p, blocks, threads, parts, v, stream);
    }
  }
  const int threads = 128;
  const size_t smem = ((size_t)p.width + (size_t)p.S * threads) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  static size_t configured = 0;
  if (smem > 48 * 1024 && smem > configured) {
    if (cudaFuncSetAttribute(stream_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return -2;
    configured = smem;
  }
  si_launch(stream_norm_kernel<T>, dim3(p.num_rows), dim3(threads), smem, stream, p);
  return si_last_error();
}

// x_dtype: dtype of y and out. `dst` may be `src`. Returns 0, a CUDA error code, or -2 (size refused).
SI_EXPORT int si_stream_norm(const float* src, long long src_row, long long src_stream, float* dst, const void* y,
                             const float* mix, const float* write, const float* read, const int* rows, const void* weight,
                             int weight_dtype, void* out, int x_dtype, int num_rows, int S, int width, float eps,
                             const void* ahead, long long ahead_bytes, cudaStream_t stream) {
  if (num_rows <= 0) return 0;
  if (S < 1 || width < 1 || !out || !weight || (y && (!mix || !write)) || (rows && dst) || (dst && !y)) return -2;
  StreamArgs p{src, src_row, src_stream, dst, y, mix, write, read, rows, weight, weight_dtype == SI_BF16 ? 1 : 0, out,
               S, width, num_rows, eps, ahead, ahead_bytes, 0};
  return x_dtype == SI_BF16 ? stream_launch<__nv_bfloat16>(p, stream) : stream_launch<float>(p, stream);
}
