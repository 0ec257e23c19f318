// What stands between a stacked q/k/v projection and attention over the paged cache when q, k and v pass a short causal
// convolution over time first:
//   row = [ q: NQ vectors of dk | k: NK vectors of dk | v: NV vectors of dv ]     (C channels in all)
//   p[t, c] = row[t, c] + bias[c]                                                  (bias absent: none)
//   y[t, c] = sum_j w[j, c] * p[t - K + 1 + j, c]                                  K taps, p = 0 before the sequence's start
//   q, k: y <- y * rsqrt(mean over the vector of y^2 + eps) (* weight)             (norm off: as it is)
//   q into `q_out`; k and v into their pages [pages, NK or NV, page_size, size].
// A layer that reads another layer's cache has NK = NV = 0: the queries alone.
// Per request the slot of the state keeps the last K - 1 values p of every channel, [K - 1, C] fp32, oldest first; a
// portion starts from them (from zeros at position 0) and leaves its own behind, so a sequence may be cut anywhere. The slot
// of a sequence that brings one row (decode) is renewed by the threads that read it, that of a sequence from its start by the
// threads of its last row (nobody reads the old values); the other portions' by a second small launch, since other blocks
// read the old values.// All arithmetic is fp32.
//
// Two further forms:
//   rotation  q and k are turned by their row's position between the convolution and the norm: the neighbouring pairs (2i, 2i + 1) of
//             a vector's first `rot_dims` entries by position * inv_freq[i]. A block makes the sines of the rows at hand once, in
//             shared memory, for all of its vectors.
//   rows      (what stands before a recurrence) y <- silu(y + out_bias) where asked, q and k unit vectors, y * rsqrt(sum(y^2) + eps)
//             (q times `q_scale`), and everything goes into fp32 rows [T, C] instead of `q_out` and pages; a second copy in
//             the compute dtype, vector by vector [vector][T][copy_size], feeds a product per vector.
//
// The fast kernel: a thread holds eight neighbouring channels (16 bytes of bfloat16) with their taps, their last K - 1
// inputs and their bias in registers and walks a few dozen rows (prompts; one row in decode steps), so that every input and
// tap is read once; the threads of a vector (a group of 2^n lanes) add their squares with shuffles. Sizes that are no multiples of 8, vectors above 256
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
  const float* inv_freq; int rot_dims;                   // rotation: fp32 [rot_dims / 2] or null
  float* rows_out; long long rows_stride;                // rows: fp32 [T, C] or null
  int silu; const float* out_bias; float q_scale;        // rows only
  void* copy; long long copy_vec; int copy_size;         // rows only: entries between vectors and between rows of the copy, or null
  int lanes_qk, rows_per_block, trigger;                 // fast kernel: lanes a q or k vector, rows a block walks
  int state_from_start;                                  // second launch: portions from position 0 as well (plain kernel)
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

// What a row needs beside its channels: looked up once by a thread each and shared by the block.
struct ConvRow {
  int seq, leaves, page, at;                             // seq -1: nothing to do; it renews the slot; its page (-1: no store), place there
  int back, pos;                                         // rows of its portion before it
  float* state;                                          // its sequence's slot
};
#define CONV_FROM_START 1
#define CONV_CONTINUED 2
#define CONV_ROWS 128                                    // most rows a block walks
#define CONV_PLAIN 0                                     // forms of the fast kernel
#define CONV_ROTATE 1
#define CONV_TO_ROWS 2
#define CONV_MAX_PAIRS 128                               // rotation in the fast kernel: pairs of a vector (of 256 entries at most)

// R: 1 (a block has one row) or 4 (it walks rows_per_block rows, the loads of four of them in flight together). The last
// values of the thread's channels stand in a ring of four, the row's place in it being a compile-time number, in pairs for
// the packed fp32 instructions.
template <typename T, int K, int R, int FORM>
__global__ void __launch_bounds__(256, 2) qkv_conv_vec_kernel(const ConvArgs p) {
  static_assert(K >= 1 && K <= 4 && (R == 1 || R == 4), "");
  constexpr int PACK = (int)sizeof(T) / 2;               // 16-byte pieces that hold eight channels
  constexpr bool STAGED = R > 1 && PACK == 1;            // rows come through shared memory, four rows ahead of the sums
  __shared__ ConvRow rows[R == 1 ? 1 : CONV_ROWS];
  __shared__ uint4 stage[STAGED ? 2 * R * 256 : 1];      // [half][row][thread]: every thread reads what it fetched itself
  __shared__ float2 turn[FORM == CONV_ROTATE ? 2 * R * CONV_MAX_PAIRS : 1];      // [half][row][pair]: cosine and sine
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
  const bool is_v = id >= qk_threads, is_q = !is_v && vec < p.NQ;
  const bool on = c >= 0;
  const bool norm = !is_v && p.norm;
  // the lanes of this thread's vector
  const unsigned group = p.lanes_qk >= 32 ? 0xffffffffu : ((1u << p.lanes_qk) - 1u) << (lane & ~(p.lanes_qk - 1));
  float2 w[K][4], b[4], ring[4][4];
#pragma unroll
  for (int e = 0; e < 4; ++e) b[e] = make_float2(0.f, 0.f);
  auto load_pairs = [](const float* src, float2 (&v)[4]) {
    const float4 lo = *reinterpret_cast<const float4*>(src), hi = *reinterpret_cast<const float4*>(src + 4);
    v[0] = make_float2(lo.x, lo.y); v[1] = make_float2(lo.z, lo.w);
    v[2] = make_float2(hi.x, hi.y); v[3] = make_float2(hi.z, hi.w);
  };
  if (on) {                                              // weights: read before the wait for the kernel before this one
#pragma unroll
    for (int j = 0; j < K; ++j) load_pairs(p.w + (size_t)j * p.C + c, w[j]);
    if (p.bias) load_pairs(p.bias + c, b);
  }
  const float* gw = !norm ? nullptr : is_q ? p.q_w : p.k_w;
  const int t0 = blockIdx.x * p.rows_per_block, nrows = min(p.rows_per_block, p.num_tokens - t0);
  if (threadIdx.x < nrows) {                             // the step's integers: copied in before any of its kernels began
    const int t = t0 + threadIdx.x;
    ConvRow r;
    r.seq = p.row_seq[t];
    r.pos = p.positions[t];
    r.back = r.leaves = r.at = 0;
    r.page = -1;
    r.state = nullptr;
    if (r.seq >= p.num_seqs) {
      set_status(p.status, SI_BAD_SEQ);
      r.seq = -1;
    }
    if (r.seq >= 0) {
      const int start = p.q_start[r.seq];
      r.back = t - start;
      const int end = p.q_start[r.seq + 1];
      r.leaves = end - start == 1 || (t == end - 1 && r.pos == r.back);
      if (p.state) r.state = p.state + (size_t)p.slots[r.seq] * p.state_stride;
      if (p.k_cache) { r.page = (int)conv_page(p, r.seq, r.pos, true); r.at = r.pos % p.page_size; }
    }
    rows[threadIdx.x] = r;
  }
  if (p.trigger) pdl_trigger();
  __syncthreads();
  pdl_wait();
  const T* u = (const T*)p.u + (size_t)t0 * p.u_stride + c;
  T* qo = (T*)p.q_out + (size_t)t0 * p.q_out_stride + c;
  auto unpack = [](const uint4* src, float2 (&v)[4]) {
    float f[8];
    load8<T>(reinterpret_cast<const T*>(src), f);
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = make_float2(f[2 * e], f[2 * e + 1]);
  };
  float2 ob[4];                                          // what is added behind the convolution
#pragma unroll
  for (int e = 0; e < 4; ++e) ob[e] = make_float2(0.f, 0.f);
  if (FORM == CONV_TO_ROWS && p.out_bias && on) load_pairs(p.out_bias + c, ob);
  // row r of the four at hand: its values join the ring, y = the convolution; returns the sum of y^2
  auto sums = [&](int r, int half, const uint4* raw, float2 (&y)[4]) {
    float2 (&x)[4] = ring[r & 3];
    if (STAGED) {
      const uint4 mine = stage[(half * R + r) * 256 + threadIdx.x];
      unpack(&mine, x);
    } else {
      unpack(raw + r * PACK, x);
    }
    float2 s2 = make_float2(0.f, 0.f);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      x[e] = __fadd2_rn(x[e], b[e]);
      y[e] = __fmul2_rn(w[0][e], ring[(r - K + 1) & 3][e]);
#pragma unroll
      for (int j = 1; j < K; ++j) y[e] = __ffma2_rn(w[j][e], ring[(r - K + 1 + j) & 3][e], y[e]);
      if (FORM == CONV_TO_ROWS) {
        y[e] = __fadd2_rn(y[e], ob[e]);
        if (p.silu) y[e] = make_float2(y[e].x / (1.f + expf(-y[e].x)), y[e].y / (1.f + expf(-y[e].y)));
      }
      s2 = __ffma2_rn(y[e], y[e], s2);
    }
    return s2.x + s2.y;
  };
  // rows take the sum of the squares, the other forms their mean
  const float inv_dk = FORM == CONV_TO_ROWS ? 1.f : 1.f / (float)p.dk;
  const float after = FORM == CONV_TO_ROWS && is_q ? p.q_scale : 1.f;
  const int pairs = FORM == CONV_ROTATE ? p.rot_dims / 2 : 0;
  auto turn_row = [&](int half, int r, float2 (&y)[4]) {       // row r of the four at hand
    if constexpr (FORM == CONV_ROTATE) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = off / 2 + e;
        if (!is_v && i < pairs) {
          const float2 cs = turn[(half * R + r) * CONV_MAX_PAIRS + i];
          y[e] = make_float2(y[e].x * cs.x - y[e].y * cs.y, y[e].y * cs.x + y[e].x * cs.y);
        }
      }
    }
  };
  auto normalise = [&](float ss, float2 (&y)[4]) {       // ss: over the whole vector
    const float inv = rsqrtf(fmaf(ss, inv_dk, p.eps)) * after;
#pragma unroll
    for (int e = 0; e < 4; ++e) y[e] = __fmul2_rn(y[e], make_float2(inv, inv));
    if (gw && on) {
      float2 g[4];
      load_pairs(gw + off, g);
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = __fmul2_rn(y[e], g[e]);
    }
  };
  // where this thread's entries of a row go: q by rows, k and v by page and place in it
  const int heads = is_v ? p.NV : p.NK, size = is_v ? p.dv : p.dk, head = is_v ? vec : vec - p.NQ;
  const long long page_step = (long long)heads * p.page_size * size;
  T* kv = is_q ? nullptr : (is_v ? (T*)p.v_cache : (T*)p.k_cache);
  if (kv) kv += (long long)head * p.page_size * size + off;
  auto put = [&](int i, const float2 (&y)[4]) {
    T* dst;
    if (FORM == CONV_TO_ROWS) {
      const float v[8] = {y[0].x, y[0].y, y[1].x, y[1].y, y[2].x, y[2].y, y[3].x, y[3].y};
      store8<float>(p.rows_out + (size_t)(t0 + i) * p.rows_stride + c, v);
      if (p.copy) store8<T>((T*)p.copy + ((is_v ? p.NQ + p.NK : 0) + vec) * p.copy_vec + (size_t)(t0 + i) * p.copy_size + off, v);
      return;
    }
    if (is_q) {
      dst = qo + (size_t)i * p.q_out_stride;
    } else {
      if (!kv || rows[i].page < 0) return;
      dst = kv + rows[i].page * page_step + rows[i].at * size;
    }
    const float out[8] = {y[0].x, y[0].y, y[1].x, y[1].y, y[2].x, y[2].y, y[3].x, y[3].y};
    store8<T>(dst, out);
  };
  auto fetch = [&](int i0, int half) {
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (on && i0 + r < nrows)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(
            &stage[(half * R + r) * 256 + threadIdx.x])), "l"(u + (size_t)(i0 + r) * p.u_stride));
    asm volatile("cp.async.commit_group;\n" ::);
  };
  if (STAGED) fetch(0, 0);
  int seq_before = -1;
  for (int i0 = 0; i0 < nrows; i0 += R) {
    uint4 raw[STAGED ? 1 : R * PACK];                    // the thread's channels of R rows
    const int half = (i0 / R) & 1;
    if constexpr (FORM == CONV_ROTATE) {                 // the rows' sines; the other half is still being read by slower warps
      for (int idx = threadIdx.x; idx < R * pairs; idx += blockDim.x) {
        const int r = idx / pairs, i = idx - r * pairs;
        if (i0 + r < nrows) {
          float sn, cs;
          sincosf((float)rows[i0 + r].pos * p.inv_freq[i], &sn, &cs);
          turn[(half * R + r) * CONV_MAX_PAIRS + i] = make_float2(cs, sn);
        }
      }
      __syncthreads();
    }
    if (STAGED) {
      fetch(i0 + R, half ^ 1);
      asm volatile("cp.async.wait_group 1;\n" ::: "memory");      // the rows at i0 have arrived
    }
#pragma unroll
    for (int r = 0; r < R && !STAGED; ++r)
      if (on && i0 + r < nrows) {
#pragma unroll
        for (int h = 0; h < PACK; ++h) raw[r * PACK + h] = reinterpret_cast<const uint4*>(u + (size_t)(i0 + r) * p.u_stride)[h];
      }
    if (R > 1) {
      // four rows that go on from the row before them, none of which renews the slot: in pairs, so that their sums overlap
      bool run = i0 + R <= nrows && seq_before >= 0;
#pragma unroll
      for (int r = 0; r < R; ++r) run = run && rows[i0 + r].seq == seq_before && !rows[i0 + r].leaves;
      if (run) {
#pragma unroll
        for (int r = 0; r < R; r += 2) {                 // two at a time: what the registers hold
          float2 y0[4], y1[4];
          float s0 = 0.f, s1 = 0.f;
          if (on) {
            s0 = sums(r, half, raw, y0);
            s1 = sums(r + 1, half, raw, y1);
            turn_row(half, r, y0);
            turn_row(half, r + 1, y1);
          }
          if (norm) {
            for (int o = 1; o < p.lanes_qk; o <<= 1) {
              s0 += __shfl_xor_sync(group, s0, o);
              s1 += __shfl_xor_sync(group, s1, o);
            }
            normalise(s0, y0);
            normalise(s1, y1);
          }
          if (on) {
            put(i0 + r, y0);
            put(i0 + r + 1, y1);
          }
        }
        continue;
      }
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = i0 + r;
      if (i >= nrows) break;
      const int seq = rows[i].seq;
      if (K > 1 && on && seq >= 0 && seq != seq_before) {          // the block's first row, or a sequence's: its past
        const int pos = rows[i].pos, back = rows[i].back;
        const float* st = rows[i].state + c;
#pragma unroll
        for (int d = 1; d < K; ++d) {                    // d rows back
          float2 (&h)[4] = ring[(r - d) & 3];
          if (d > pos) {
#pragma unroll
            for (int e = 0; e < 4; ++e) h[e] = make_float2(0.f, 0.f);
          } else if (d <= back) {
            uint4 old[PACK];
#pragma unroll
            for (int q = 0; q < PACK; ++q) old[q] = reinterpret_cast<const uint4*>(u + (ptrdiff_t)(i - d) * p.u_stride)[q];
            unpack(old, h);
#pragma unroll
            for (int e = 0; e < 4; ++e) h[e] = __fadd2_rn(h[e], b[e]);
          } else {
            load_pairs(st + (size_t)(K - 1 - (d - back)) * p.C, h);
          }
        }
      }
      seq_before = seq;
      if (seq < 0) continue;                             // a padding row of a fixed-shape step, or a fault
      float2 y[4];
      float ss = 0.f;
      if (on) {
        ss = sums(r, half, raw, y);
        turn_row(half, r, y);
        if (K > 1 && rows[i].leaves) {                   // nobody else reads or writes its slot in this launch
#pragma unroll
          for (int d = 0; d < K - 1; ++d) {
            const float2 (&h)[4] = ring[(r - d) & 3];
            float* dst = rows[i].state + (size_t)(K - 2 - d) * p.C + c;
            *reinterpret_cast<float4*>(dst) = make_float4(h[0].x, h[0].y, h[1].x, h[1].y);
            *reinterpret_cast<float4*>(dst + 4) = make_float4(h[2].x, h[2].y, h[3].x, h[3].y);
          }
        }
      }
      if (norm) {                                        // whole groups of lanes are q and k, or not
        for (int o = 1; o < p.lanes_qk; o <<= 1) ss += __shfl_xor_sync(group, ss, o);
        normalise(ss, y);
      }
      if (on) put(i, y);
    }
  }
}

template <typename T, int R, int FORM>
static void conv_launch_vec(ConvArgs& p, int yb, int threads, cudaStream_t stream) {
  p.rows_per_block = 1;
  if (R > 1) {                                           // as many rows as let all blocks run at once (two a multiprocessor)
    const long long blocks = 2LL * si_sm_count() / yb > 0 ? 2LL * si_sm_count() / yb : 1;
    const long long per = (p.num_tokens + blocks - 1) / blocks;
    p.rows_per_block = (int)(per > CONV_ROWS ? CONV_ROWS : (per + R - 1) / R * R);
  }
  const dim3 grid((p.num_tokens + p.rows_per_block - 1) / p.rows_per_block, yb);
  p.trigger = si_pdl_trigger_mode((long long)grid.x * grid.y, 2LL * si_sm_count()) == 1;
  switch (p.K) {
    case 1: si_launch(qkv_conv_vec_kernel<T, 1, R, FORM>, grid, dim3(threads), 0, stream, p); break;
    case 2: si_launch(qkv_conv_vec_kernel<T, 2, R, FORM>, grid, dim3(threads), 0, stream, p); break;
    case 3: si_launch(qkv_conv_vec_kernel<T, 3, R, FORM>, grid, dim3(threads), 0, stream, p); break;
    default: si_launch(qkv_conv_vec_kernel<T, 4, R, FORM>, grid, dim3(threads), 0, stream, p); break;
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
    if (p.out_bias) y += p.out_bias[c];
    return p.silu ? y / (1.f + expf(-y)) : y;
  };
  // entry i of this warp's vector, turned where the vector is a query or key and the entry lies among those that are
  auto entry = [&](int i) {
    const float y = value(c0 + i);
    if (is_v || !p.inv_freq || i >= p.rot_dims) return y;
    const float other = value(c0 + (i ^ 1));
    float sn, cs;
    sincosf((float)pos * p.inv_freq[i / 2], &sn, &cs);
    return (i & 1) ? y * cs + other * sn : y * cs - other * sn;
  };
  float inv = 1.f;
  if (!is_v && p.norm) {
    float ss = 0.f;
    for (int i = lane; i < size; i += 32) { const float y = value(c0 + i); ss = fmaf(y, y, ss); }
    inv = p.rows_out ? rsqrtf(warp_sum(ss) + p.eps) * (vec < p.NQ ? p.q_scale : 1.f) : rsqrtf(warp_sum(ss) / (float)size + p.eps);
  }
  T* dst = nullptr;
  if (p.rows_out) {
    // nothing but the rows
  } else if (!is_v && vec < p.NQ) {
    dst = (T*)p.q_out + (size_t)t * p.q_out_stride + c0;
  } else if (p.k_cache) {
    const long long page = conv_page(p, seq, pos, lane == 0);
    const int at = pos % p.page_size;
    if (page >= 0) dst = is_v ? (T*)p.v_cache + (((size_t)page * p.NV + (vec - p.NQ - p.NK)) * p.page_size + at) * p.dv
                              : (T*)p.k_cache + (((size_t)page * p.NK + (vec - p.NQ)) * p.page_size + at) * p.dk;
  }
  const float* gw = (is_v || !p.norm) ? nullptr : (vec < p.NQ ? p.q_w : p.k_w);
  const bool alone = p.q_start[seq + 1] - start == 1;
  // a turned entry reads its neighbour's past, so the slot moves on only when all of them have been formed
  const bool two = alone && K > 1 && p.inv_freq && !is_v;
  for (int i = lane; i < size; i += 32) {
    const float y = entry(i) * inv;
    if (p.rows_out) {
      p.rows_out[(size_t)t * p.rows_stride + c0 + i] = y;
      if (p.copy) ((T*)p.copy)[vec * p.copy_vec + (size_t)t * p.copy_size + i] = from_f32<T>(y);
    }
    if (dst) dst[i] = from_f32<T>(gw ? y * gw[i] : y);
    if (alone && K > 1 && !two) {                        // the slot moves on by one row (this lane alone reads this channel)
      float* sc = st + c0 + i;
      for (int j = 0; j + 1 < K - 1; ++j) sc[(size_t)j * p.C] = pos > 0 ? sc[(size_t)(j + 1) * p.C] : 0.f;
      sc[(size_t)(K - 2) * p.C] = to_f32<T>(u[(size_t)t * p.u_stride + c0 + i]) + (p.bias ? p.bias[c0 + i] : 0.f);
    }
  }
  if (!two) return;
  __syncwarp();
  for (int i = lane; i < size; i += 32) {
    float* sc = st + c0 + i;
    for (int j = 0; j + 1 < K - 1; ++j) sc[(size_t)j * p.C] = pos > 0 ? sc[(size_t)(j + 1) * p.C] : 0.f;
    sc[(size_t)(K - 2) * p.C] = to_f32<T>(u[(size_t)t * p.u_stride + c0 + i]) + (p.bias ? p.bias[c0 + i] : 0.f);
  }
}

// The slots of the sequences that brought more than one row: the last K - 1 values of every channel. One thread a
// (sequence, channel); entry i is the value at row n - K + 1 + i of the portion, an old entry where that lies before it.
template <typename T>
__global__ void qkv_conv_state_kernel(const ConvArgs p) {
  const int s = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= p.C) return;
  // the step's integers and the weights do not depend on the kernel before this one
  const int row0 = p.q_start[s], n = p.q_start[s + 1] - row0;
  const int pos0 = p.ctx_len[s] - n, H = p.K - 1;
  const float b = p.bias ? p.bias[c] : 0.f;
  const T* u = (const T*)p.u;
  float* st = p.state + (size_t)p.slots[s] * p.state_stride + c;
  pdl_wait();
  if (n <= 1 || (pos0 == 0 && !p.state_from_start)) return;
  auto entry = [&](int i) {
    const int r = n - H + i;
    if (r >= 0) return to_f32<T>(u[(size_t)(row0 + r) * p.u_stride + c]) + b;
    return pos0 + r < 0 ? 0.f : st[(size_t)(H + r) * p.C];
  };
  if (H <= 4) {                                          // all loads before the first store
    float x[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) x[i] = i < H ? entry(i) : 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (i < H) st[(size_t)i * p.C] = x[i];
    return;
  }
  for (int i = 0; i < H; ++i) st[(size_t)i * p.C] = entry(i);      // in order: an entry is read before a later turn overwrites it
}

template <typename T>
static int conv_launch(ConvArgs p, int portions, int* launches, cudaStream_t stream) {
  const auto al = [](const void* q) { return ((uintptr_t)q % 16) == 0; };
  const int elem = 16 / (int)sizeof(T);
  bool vec = p.K <= 4 && p.dk % 8 == 0 && p.dk <= 256 && (p.NV == 0 || p.dv % 8 == 0) && p.u_stride % elem == 0 &&
             p.q_out_stride % elem == 0 && p.state_stride % 4 == 0 && al(p.u) && al(p.bias) && al(p.w) && al(p.state) && al(p.k_cache) &&
             al(p.v_cache) && al(p.q_out) && al(p.q_w) && al(p.k_w);
  const int form = p.rows_out ? CONV_TO_ROWS : p.inv_freq ? CONV_ROTATE : CONV_PLAIN;
  if (form == CONV_TO_ROWS) vec = vec && al(p.rows_out) && p.rows_stride % 4 == 0 && al(p.out_bias) && al(p.copy) && p.copy_vec % elem == 0 && p.copy_size % elem == 0;
  if (vec) {
    p.lanes_qk = 1;
    while (p.lanes_qk * 8 < p.dk) p.lanes_qk *= 2;
    const long long want = (long long)(p.NQ + p.NK) * p.lanes_qk + (long long)p.NV * p.dv / 8;
    const int threads = want <= 128 ? 128 : 256;
    const int yb = (int)((want + threads - 1) / threads);
    // a row a block while all of them run at once, else several rows whose loads overlap
    const bool few = (long long)p.num_tokens * yb <= 2LL * si_sm_count();
    if (form == CONV_TO_ROWS) {
      if (few) conv_launch_vec<T, 1, CONV_TO_ROWS>(p, yb, threads, stream);
      else conv_launch_vec<T, 4, CONV_TO_ROWS>(p, yb, threads, stream);
    } else if (form == CONV_ROTATE) {
      if (few) conv_launch_vec<T, 1, CONV_ROTATE>(p, yb, threads, stream);
      else conv_launch_vec<T, 4, CONV_ROTATE>(p, yb, threads, stream);
    } else {
      if (few) conv_launch_vec<T, 1, CONV_PLAIN>(p, yb, threads, stream);
      else conv_launch_vec<T, 4, CONV_PLAIN>(p, yb, threads, stream);
    }
  } else {
    const dim3 grid(p.num_tokens, (p.NQ + p.NK + p.NV + 3) / 4);
    si_launch(qkv_conv_kernel<T>, grid, dim3(128), 0, stream, p);
    p.state_from_start = 1;
  }
  if (launches) *launches = 1;
  if (p.K > 1 && (portions & (vec ? CONV_CONTINUED : CONV_CONTINUED | CONV_FROM_START))) {
    if (launches) *launches = 2;
    si_launch(qkv_conv_state_kernel<T>, dim3((p.C + 127) / 128, p.num_seqs), dim3(128), 0, stream, p);
  }
  return si_last_error();
}

static bool conv_sizes_ok(const ConvArgs& p, long long C) {
  return p.NQ >= 0 && p.NK >= 0 && p.NV >= 0 && p.dk > 0 && p.dv >= 0 && p.K >= 1 && p.num_seqs <= 65535 && !(p.K > 1 && !p.state) &&
         C <= (1LL << 30) && !(p.K > 1 && p.state_stride < (long long)(p.K - 1) * C);
}

// `portions`: what the step holds beside sequences of one row: 1 portions of several rows that begin at position 0, 2 such
// portions that begin later, 3 both (or not known); 0 neither (a decode step). `launches` (may be null): kernels launched.
// `inv_freq` (fp32 [rot_dims / 2], may be null): q and k are turned in neighbouring pairs before the norm.
// Returns 0, a CUDA error code, or -2 (size refused).
SI_EXPORT int si_qkv_conv(const void* u, int dtype, long long u_stride, const float* bias, const float* w, float* state,
                          long long state_stride, const int* positions, const int* row_seq, const int* q_start,
                          const int* ctx_len, const int* slots, const int* block_table, int table_width, void* k_cache,
                          void* v_cache, int num_pages, int page_size, int num_tokens, int num_seqs, int NQ, int NK, int NV,
                          int dk, int dv, int K, void* q_out, long long q_out_stride, int norm, const float* q_w,
                          const float* k_w, float eps, const float* inv_freq, int rot_dims, int portions, int* launches, int* status,
                          cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  const long long C = (long long)(NQ + NK) * dk + (long long)NV * dv;
  if ((NK > 0 || NV > 0) && k_cache && (!block_table || page_size <= 0 || (NV > 0 && !v_cache))) return -2;
  if (inv_freq && (rot_dims < 0 || rot_dims % 2 || rot_dims > dk)) return -2;
  ConvArgs p = {};
  p.u = u; p.u_stride = u_stride; p.bias = bias; p.w = w; p.state = state; p.state_stride = state_stride;
  p.positions = positions; p.row_seq = row_seq; p.q_start = q_start; p.ctx_len = ctx_len; p.slots = slots;
  p.block_table = block_table; p.table_width = table_width; p.k_cache = k_cache; p.v_cache = v_cache;
  p.num_pages = num_pages; p.page_size = page_size; p.num_tokens = num_tokens; p.num_seqs = num_seqs;
  p.NQ = NQ; p.NK = NK; p.NV = NV; p.dk = dk; p.dv = dv; p.C = (int)C; p.K = K; p.q_out = q_out; p.q_out_stride = q_out_stride;
  p.norm = norm; p.q_w = q_w; p.k_w = k_w; p.eps = eps; p.inv_freq = rot_dims > 0 ? inv_freq : nullptr; p.rot_dims = rot_dims;
  p.q_scale = 1.f; p.lanes_qk = 1; p.rows_per_block = 1; p.status = status;
  if (!conv_sizes_ok(p, C)) return -2;
  return dtype == SI_BF16 ? conv_launch<__nv_bfloat16>(p, portions, launches, stream) : conv_launch<float>(p, portions, launches, stream);
}

// The form that leaves fp32 rows (see the head of this file): rows_out [T, C]; `unit`: q and k become unit vectors
// (x * rsqrt(sum(x^2) + eps), q times q_scale); `silu` and `out_bias` (fp32 [C], may be null) behind the convolution; `copy`
// (may be null): vector v of row t at copy + v * copy_vec + t * copy_size, in the compute dtype.
SI_EXPORT int si_conv_rows(const void* u, int dtype, long long u_stride, const float* bias, const float* w, float* state,
                           long long state_stride, const int* positions, const int* row_seq, const int* q_start,
                           const int* ctx_len, const int* slots, int num_tokens, int num_seqs, int NQ, int NK, int NV, int dk, int dv,
                           int K, float* rows_out, long long rows_stride, int unit, float eps, float q_scale, int silu,
                           const float* out_bias, void* copy, long long copy_vec, int copy_size, int portions, int* launches,
                           int* status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  const long long C = (long long)(NQ + NK) * dk + (long long)NV * dv;
  if (!rows_out || rows_stride < C) return -2;
  ConvArgs p = {};
  p.u = u; p.u_stride = u_stride; p.bias = bias; p.w = w; p.state = state; p.state_stride = state_stride;
  p.positions = positions; p.row_seq = row_seq; p.q_start = q_start; p.ctx_len = ctx_len; p.slots = slots;
  p.page_size = 1; p.num_tokens = num_tokens; p.num_seqs = num_seqs;
  p.NQ = NQ; p.NK = NK; p.NV = NV; p.dk = dk; p.dv = dv; p.C = (int)C; p.K = K;
  p.norm = unit; p.eps = eps; p.rows_out = rows_out; p.rows_stride = rows_stride; p.silu = silu; p.out_bias = out_bias;
  p.q_scale = q_scale; p.copy = copy; p.copy_vec = copy_vec; p.copy_size = copy_size;
  p.lanes_qk = 1; p.rows_per_block = 1; p.status = status;
  if (!conv_sizes_ok(p, C)) return -2;
  return dtype == SI_BF16 ? conv_launch<__nv_bfloat16>(p, portions, launches, stream) : conv_launch<float>(p, portions, launches, stream);
}
