// What stands between a stacked q/k/v projection and attention over the paged cache when q, k and v pass a short causal
// convolution over time first:
//   row = [ q: NQ vectors of dk | k: NK vectors of dk | v: NV vectors of dv ]     (C channels in all)
//   p[t, c] = row[t, c] + bias[c]                                                  (bias absent: none)
//   y[t, c] = sum_j w[j, c] * p[t - K + 1 + j, c]                                  K taps, p = 0 before the sequence's start
//   q, k: y <- y * rsqrt(mean over the vector of y^2 + eps) (* weight)             (norm off: as it is)
//   q into `q_out`; k and v into their pages [pages, NK or NV, page_size, size].
// A layer that reads another layer's cache has NK = NV = 0: the queries alone.
// Per request the slot of the state keeps the last K - 1 values p of every channel, [K - 1, C] fp32, oldest first; a
// portion starts from them (from zeros at position 0) and leaves its own behind, so a sequence may be cut anywhere. A
// sequence that brings one row (decode) has its slot renewed by the thread that read it; longer portions by a second small
// launch, since other blocks read the old values. All arithmetic is fp32.
//
// The fast kernel: a thread holds eight neighbouring channels (16 bytes of bfloat16) with their taps, their last K - 1
// inputs and their bias in registers and walks up to a few dozen rows, so that every input is read once; the threads of a
// vector (a group of 2^n lanes) add their squares with shuffles. Sizes that are no multiples of 8, vectors above 256
// entries and more than four taps take the plain kernel: a warp a vector, every tap read where it lies.
#include "common.cuh"

struct ConvArgs {
  const void* u; long long u_stride;
  const float* bias; const float* w;                     // [C]; [K, C]
  float* state; long long state_stride;
  const int* positions; const int* row_seq; const int* q_start; const int* ctx_len; const int* slots;
  const int* block_table; int table_width;
  void* k_cache; void* v_cache;
  int num_pages, page_size, num_tokens, num_seqs, NQ, NK, NV, dk, dv, C, K;
  void* q_out; long long q_out_stride;
  int norm; const float* q_w; const float* k_w; float eps;
  int rows_per_block, lanes_qk, trigger;                 // fast kernel: rows a block walks, lanes a q or k vector
  int* status;
};

template <typename T> __device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <> __device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <> __device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(h[i]);
    v[2 * i] = f.x; v[2 * i + 1] = f.y;
  }
}
template <typename T> __device__ __forceinline__ void store8(T* p, const float (&v)[8]);
template <> __device__ __forceinline__ void store8<float>(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
template <> __device__ __forceinline__ void store8<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 raw;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = raw;
}

// The page of (seq, pos), or -1; `first`: the thread that reports a bad entry.
__device__ __forceinline__ long long conv_page(const ConvArgs& p, int seq, int pos, bool first) {
  const int slot = pos / p.page_size;
  const int page = (pos >= 0 && slot < p.table_width) ? p.block_table[(size_t)seq * p.table_width + slot] : -1;
  if (page < 0 || page >= p.num_pages) {
    if (first) set_status(p.status, SI_BAD_PAGE);
    return -1;
  }
  return page;
}

template <typename T, int K>
__global__ void __launch_bounds__(256) qkv_conv_vec_kernel(const ConvArgs p) {
  constexpr int HIST = K > 1 ? K - 1 : 1;
  const int lane = threadIdx.x & 31;
  const int id = blockIdx.y * blockDim.x + threadIdx.x;
  // threads of the q and k vectors first (lanes_qk each, those beyond dk / 8 idle), then one for every 8 channels of v
  const int qk_threads = (p.NQ + p.NK) * p.lanes_qk;
  int c = -1, vec = 0, off = 0;                          // first channel of this thread (-1: none), its vector, place in it
  if (id < qk_threads) {
    vec = id / p.lanes_qk;
    off = (id % p.lanes_qk) * 8;
    if (off < p.dk) c = vec * p.dk + off;
  } else if (p.NV > 0) {
    const int e = (id - qk_threads) * 8;
    if (e < p.NV * p.dv) { vec = e / p.dv; off = e % p.dv; c = (p.NQ + p.NK) * p.dk + e; }
  }
  const bool is_v = id >= qk_threads;
  const bool on = c >= 0;
  // the lanes of this thread's vector
  const unsigned group = p.lanes_qk >= 32 ? 0xffffffffu : ((1u << p.lanes_qk) - 1u) << (lane & ~(p.lanes_qk - 1));
  float w[K][8], b[8], g[8], hist[HIST][8];              // hist[j]: the value j + 1 rows back
#pragma unroll
  for (int e = 0; e < 8; ++e) { b[e] = 0.f; g[e] = 1.f; }
  if (on) {                                              // weights: read before the wait for the kernel before this one
#pragma unroll
    for (int j = 0; j < K; ++j) load8<float>(p.w + (size_t)j * p.C + c, w[j]);
    if (p.bias) load8<float>(p.bias + c, b);
    if (!is_v && p.norm) {
      const float* gw = vec < p.NQ ? p.q_w : p.k_w;
      if (gw) load8<float>(gw + off, g);
    }
  }
  if (p.trigger) pdl_trigger();
  pdl_wait();
  const T* u = (const T*)p.u;
  const int t0 = blockIdx.x * p.rows_per_block, t1 = min(p.num_tokens, t0 + p.rows_per_block);
  int seq_before = -1;
  for (int t = t0; t < t1; ++t) {
    const int seq = p.row_seq[t];
    if (seq < 0 || seq >= p.num_seqs) {                  // a padding row of a fixed-shape step, or a fault
      if (seq >= 0 && id == 0) set_status(p.status, SI_BAD_SEQ);
      seq_before = -1;
      continue;
    }
    const int pos = p.positions[t];
    const int start = p.q_start[seq];
    float* st = p.state ? p.state + (size_t)p.slots[seq] * p.state_stride : nullptr;
    if (on && K > 1 && seq != seq_before) {              // the block's first row, or a sequence's first row: its past
      const int back = t - start;
#pragma unroll
      for (int j = 0; j < K - 1; ++j) {
        const int d = j + 1;                             // rows back
        if (d > pos) {
#pragma unroll
          for (int e = 0; e < 8; ++e) hist[j][e] = 0.f;
        } else if (d <= back) {
          load8<T>(u + (size_t)(t - d) * p.u_stride + c, hist[j]);
#pragma unroll
          for (int e = 0; e < 8; ++e) hist[j][e] += b[e];
        } else {
          load8<float>(st + (size_t)(K - 1 - (d - back)) * p.C + c, hist[j]);
        }
      }
    }
    seq_before = seq;
    float y[8];
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) y[e] = 0.f;
    if (on) {
      float x[8];
      load8<T>(u + (size_t)t * p.u_stride + c, x);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] += b[e];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
#pragma unroll
        for (int j = 0; j < K - 1; ++j) y[e] = fmaf(w[j][e], hist[K - 2 - j][e], y[e]);
        y[e] = fmaf(w[K - 1][e], x[e], y[e]);
        ss = fmaf(y[e], y[e], ss);
      }
      if (K > 1) {
#pragma unroll
        for (int j = HIST - 1; j > 0; --j)
#pragma unroll
          for (int e = 0; e < 8; ++e) hist[j][e] = hist[j - 1][e];
#pragma unroll
        for (int e = 0; e < 8; ++e) hist[0][e] = x[e];
        if (p.q_start[seq + 1] - start == 1) {           // the sequence's only row: nobody else reads or writes its slot here
#pragma unroll
          for (int j = 0; j < K - 1; ++j) store8<float>(st + (size_t)(K - 2 - j) * p.C + c, hist[j]);
        }
      }
    }
    if (!is_v && p.norm) {                               // whole groups of lanes are q and k, or not
      for (int o = 1; o < p.lanes_qk; o <<= 1) ss += __shfl_xor_sync(group, ss, o);
      const float inv = rsqrtf(ss / (float)p.dk + p.eps);
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] *= inv * g[e];
    }
    if (!on) continue;
    if (!is_v && vec < p.NQ) {
      store8<T>((T*)p.q_out + (size_t)t * p.q_out_stride + c, y);
    } else if (p.k_cache) {
      const long long page = conv_page(p, seq, pos, lane == 0);
      if (page < 0) continue;
      const int at = pos % p.page_size;
      if (is_v) store8<T>((T*)p.v_cache + (((size_t)page * p.NV + vec) * p.page_size + at) * p.dv + off, y);
      else store8<T>((T*)p.k_cache + (((size_t)page * p.NK + (vec - p.NQ)) * p.page_size + at) * p.dk + off, y);
    }
  }
}

// Any size: a warp a vector, a block of four vectors a row.
template <typename T>
__global__ void __launch_bounds__(128) qkv_conv_kernel(const ConvArgs p) {
  pdl_prologue();
  const int lane = threadIdx.x & 31, vec = blockIdx.y * 4 + (threadIdx.x >> 5), t = blockIdx.x;
  if (vec >= p.NQ + p.NK + p.NV) return;
  const int seq = p.row_seq[t];
  if (seq < 0 || seq >= p.num_seqs) {
    if (seq >= 0 && threadIdx.x == 0) set_status(p.status, SI_BAD_SEQ);
    return;
  }
  const bool is_v = vec >= p.NQ + p.NK;
  const int size = is_v ? p.dv : p.dk;
  const int c0 = is_v ? (p.NQ + p.NK) * p.dk + (vec - p.NQ - p.NK) * p.dv : vec * p.dk;
  const int pos = p.positions[t], start = p.q_start[seq], back = t - start, K = p.K;
  const T* u = (const T*)p.u;
  float* st = p.state ? p.state + (size_t)p.slots[seq] * p.state_stride : nullptr;
  auto value = [&](int c) {
    const float b = p.bias ? p.bias[c] : 0.f;
    float y = 0.f;
    for (int j = 0; j < K; ++j) {
      const int d = K - 1 - j;                           // rows back
      if (d > pos) continue;
      const float x = d <= back ? to_f32<T>(u[(size_t)(t - d) * p.u_stride + c]) + b : st[(size_t)(K - 1 - (d - back)) * p.C + c];
      y = fmaf(p.w[(size_t)j * p.C + c], x, y);
    }
    return y;
  };
  float inv = 1.f;
  if (!is_v && p.norm) {
    float ss = 0.f;
    for (int i = lane; i < size; i += 32) { const float y = value(c0 + i); ss = fmaf(y, y, ss); }
    inv = rsqrtf(warp_sum(ss) / (float)size + p.eps);
  }
  T* dst = nullptr;
  if (!is_v && vec < p.NQ) {
    dst = (T*)p.q_out + (size_t)t * p.q_out_stride + c0;
  } else if (p.k_cache) {
    const long long page = conv_page(p, seq, pos, lane == 0);
    const int at = pos % p.page_size;
    if (page >= 0) dst = is_v ? (T*)p.v_cache + (((size_t)page * p.NV + (vec - p.NQ - p.NK)) * p.page_size + at) * p.dv
                              : (T*)p.k_cache + (((size_t)page * p.NK + (vec - p.NQ)) * p.page_size + at) * p.dk;
  }
  const float* gw = (is_v || !p.norm) ? nullptr : (vec < p.NQ ? p.q_w : p.k_w);
  const bool alone = p.q_start[seq + 1] - start == 1;
  for (int i = lane; i < size; i += 32) {
    const float y = value(c0 + i) * inv;
    if (dst) dst[i] = from_f32<T>(gw ? y * gw[i] : y);
    if (alone && K > 1) {                                // the slot moves on by one row (this lane alone reads this channel)
      float* sc = st + c0 + i;
      for (int j = 0; j + 1 < K - 1; ++j) sc[(size_t)j * p.C] = pos > 0 ? sc[(size_t)(j + 1) * p.C] : 0.f;
      sc[(size_t)(K - 2) * p.C] = to_f32<T>(u[(size_t)t * p.u_stride + c0 + i]) + (p.bias ? p.bias[c0 + i] : 0.f);
    }
  }
}

// The slots of the sequences that brought more than one row: the last K - 1 values of every channel. One thread a
// (sequence, channel); entry i is the value at row n - K + 1 + i of the portion, an old entry where that lies before it.
template <typename T>
__global__ void qkv_conv_state_kernel(const ConvArgs p) {
  pdl_prologue();
  const int s = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= p.C) return;
  const int row0 = p.q_start[s], n = p.q_start[s + 1] - row0;
  if (n <= 1) return;
  const int pos0 = p.ctx_len[s] - n, H = p.K - 1;
  const float b = p.bias ? p.bias[c] : 0.f;
  const T* u = (const T*)p.u;
  float* st = p.state + (size_t)p.slots[s] * p.state_stride + c;
  for (int i = 0; i < H; ++i) {                          // in order: an entry is read before a later turn overwrites it
    const int r = n - H + i;
    float x;
    if (r >= 0) x = to_f32<T>(u[(size_t)(row0 + r) * p.u_stride + c]) + b;
    else if (pos0 + r < 0) x = 0.f;
    else x = st[(size_t)(H + r) * p.C];
    st[(size_t)i * p.C] = x;
  }
}

template <typename T>
static int conv_launch(ConvArgs p, int longest, cudaStream_t stream) {
  const auto al = [](const void* q) { return ((uintptr_t)q % 16) == 0; };
  const int elem = 16 / (int)sizeof(T);
  bool vec = p.K <= 4 && p.dk % 8 == 0 && p.dk <= 256 && (p.NV == 0 || p.dv % 8 == 0) && p.u_stride % elem == 0 &&
             p.q_out_stride % elem == 0 && p.state_stride % 4 == 0 && al(p.u) && al(p.bias) && al(p.w) && al(p.state) && al(p.k_cache) &&
             al(p.v_cache) && al(p.q_out) && al(p.q_w) && al(p.k_w);
  if (vec) {
    p.lanes_qk = 1;
    while (p.lanes_qk * 8 < p.dk) p.lanes_qk *= 2;
    const long long want = (long long)(p.NQ + p.NK) * p.lanes_qk + (long long)p.NV * p.dv / 8;
    const int threads = want <= 128 ? 128 : 256;
    const int yb = (int)((want + threads - 1) / threads);
    long long rows = (long long)p.num_tokens * yb / (8LL * si_sm_count());
    p.rows_per_block = rows < 1 ? 1 : (rows > 16 ? 16 : (int)rows);
    const dim3 grid((p.num_tokens + p.rows_per_block - 1) / p.rows_per_block, yb);
    p.trigger = si_pdl_trigger_mode((long long)grid.x * grid.y, 2LL * si_sm_count()) == 1 && longest == 1;
    switch (p.K) {
      case 1: si_launch(qkv_conv_vec_kernel<T, 1>, grid, dim3(threads), 0, stream, p); break;
      case 2: si_launch(qkv_conv_vec_kernel<T, 2>, grid, dim3(threads), 0, stream, p); break;
      case 3: si_launch(qkv_conv_vec_kernel<T, 3>, grid, dim3(threads), 0, stream, p); break;
      default: si_launch(qkv_conv_vec_kernel<T, 4>, grid, dim3(threads), 0, stream, p); break;
    }
  } else {
    const dim3 grid(p.num_tokens, (p.NQ + p.NK + p.NV + 3) / 4);
    si_launch(qkv_conv_kernel<T>, grid, dim3(128), 0, stream, p);
  }
  if (p.K > 1 && longest != 1)
    si_launch(qkv_conv_state_kernel<T>, dim3((p.C + 127) / 128, p.num_seqs), dim3(128), 0, stream, p);
  return si_last_error();
}

// Most rows that one call's sequence brings: `longest` (1: a decode step, no second launch; 0: not known).
// Returns 0, a CUDA error code, or -2 (size refused).
SI_EXPORT int si_qkv_conv(const void* u, int dtype, long long u_stride, const float* bias, const float* w, float* state,
                          long long state_stride, const int* positions, const int* row_seq, const int* q_start,
                          const int* ctx_len, const int* slots, const int* block_table, int table_width, void* k_cache,
                          void* v_cache, int num_pages, int page_size, int num_tokens, int num_seqs, int NQ, int NK, int NV,
                          int dk, int dv, int K, void* q_out, long long q_out_stride, int norm, const float* q_w,
                          const float* k_w, float eps, int longest, int* status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (NQ < 0 || NK < 0 || NV < 0 || dk <= 0 || dv < 0 || K < 1 || num_seqs > 65535 || (K > 1 && !state)) return -2;
  if ((NK > 0 || NV > 0) && k_cache && (!block_table || page_size <= 0 || (NV > 0 && !v_cache))) return -2;
  const long long C = (long long)(NQ + NK) * dk + (long long)NV * dv;
  if (C > (1LL << 30) || state_stride < (long long)(K - 1) * C) return -2;
  ConvArgs p{u, u_stride, bias, w, state, state_stride, positions, row_seq, q_start, ctx_len, slots, block_table, table_width,
             k_cache, v_cache, num_pages, page_size, num_tokens, num_seqs, NQ, NK, NV, dk, dv, (int)C, K, q_out, q_out_stride,
             norm, q_w, k_w, eps, 1, 1, 0, status};
  return dtype == SI_BF16 ? conv_launch<__nv_bfloat16>(p, longest, stream) : conv_launch<float>(p, longest, stream);
}
