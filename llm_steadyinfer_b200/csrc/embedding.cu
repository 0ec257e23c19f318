// Embedding gather: out[t, :] = scale * table[tokens[t], :] (or its RMS norm times a weight, all fp32), widened to fp32 (the residual
// stream is fp32 in both precisions; the product with the scale is fp32 too). The reference's kernel
// (src/source/op/kernels/cuda/emb_kernel.cu:3-21) silently skips token ids outside
// the vocabulary; here such a row is zeroed and the status word is set.
#include "common.cuh"

template <typename TW>
__global__ void embedding_gather_kernel(const int* __restrict__ tokens, const TW* __restrict__ table,
                                        float* __restrict__ out, int hidden, int vocab,
                                        float scale, const float* __restrict__ norm_w, float eps, int* status) {
  __shared__ float scratch[33];
  pdl_prologue();
  const int t = blockIdx.x;
  const int tok = tokens[t];
  float* o = out + (size_t)t * hidden;
  if (tok < 0 || tok >= vocab) {
    if (threadIdx.x == 0) set_status(status, SI_BAD_TOKEN);
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) o[i] = 0.f;
    return;
  }
  const TW* w = table + (size_t)tok * hidden;
  if (norm_w) {                              // a norm on the embedding's output, in the same launch
    float ss = 0.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
      const float x = scale * to_f32<TW>(w[i]);
      ss = fmaf(x, x, ss);
    }
    const float inv = rsqrtf(block_sum(ss, scratch) / (float)hidden + eps);
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) o[i] = norm_w[i] * (scale * to_f32<TW>(w[i]) * inv);
    return;
  }
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) o[i] = scale * to_f32<TW>(w[i]);
}

SI_EXPORT int si_embedding_gather(const int* tokens, const void* table, int table_dtype, float* out,
                                  int num_tokens, int hidden, int vocab, float scale, const float* norm_w, float eps,
                                  int* status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  const int threads = hidden >= 1024 ? 256 : 128;
  if (table_dtype == SI_BF16)
    si_launch(embedding_gather_kernel<__nv_bfloat16>, dim3(num_tokens), dim3(threads), 0, stream,
              tokens, (const __nv_bfloat16*)table, out, hidden, vocab, scale, norm_w, eps, status);
  else
    si_launch(embedding_gather_kernel<float>, dim3(num_tokens), dim3(threads), 0, stream,
              tokens, (const float*)table, out, hidden, vocab, scale, norm_w, eps, status);
  return si_last_error();
}

// Embedding plus a hashed embedding of the token pair (previous, current):
//   out[t, :] = table[tok_t, :] + pair[r_t, :]
//   r_t = (tok_{t-1} * mul_prev + tok_t * mul_cur) mod buckets,  and r = buckets (the table's extra last row)
//   for the first token of a sequence.
// The previous token of a portion's first row is what the request's state slot holds (int32, one per slot);
// the block of that row reads it and then stores the portion's last token there for the next step, so the
// sequence may be cut anywhere and a token that was sampled on the device needs no trip to the host.
template <typename TW>
__global__ void embedding_pair_kernel(const int* __restrict__ tokens, const int* __restrict__ positions,
                                      const int* __restrict__ row_seq, const int* __restrict__ q_start,
                                      const int* __restrict__ slots, int* __restrict__ last_token,
                                      const TW* __restrict__ table, const TW* __restrict__ pair,
                                      float* __restrict__ out, int hidden, int vocab, int buckets,
                                      long long mul_prev, long long mul_cur, int num_seqs, int* status) {
  __shared__ int s_prev;
  pdl_prologue();
  const int t = blockIdx.x;
  const int tok = tokens[t];
  const int seq = row_seq[t];
  float* o = out + (size_t)t * hidden;
  if (seq < 0 || seq >= num_seqs || tok < 0 || tok >= vocab) {
    if (threadIdx.x == 0 && seq >= 0) set_status(status, seq >= num_seqs ? SI_BAD_SEQ : SI_BAD_TOKEN);
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) o[i] = 0.f;
    return;
  }
  if (threadIdx.x == 0) {
    const int row0 = q_start[seq];
    int prev;
    if (t > row0) {
      prev = tokens[t - 1];
    } else {
      int* slot = last_token + slots[seq];
      prev = *slot;
      *slot = tokens[q_start[seq + 1] - 1];           // what the next step's first row pairs with
    }
    s_prev = prev;
  }
  __syncthreads();
  long long r = buckets;
  if (positions[t] > 0) {
    const int prev = s_prev;
    if (prev < 0 || prev >= vocab) {
      if (threadIdx.x == 0) set_status(status, SI_BAD_TOKEN);
      for (int i = threadIdx.x; i < hidden; i += blockDim.x) o[i] = 0.f;
      return;
    }
    r = ((long long)prev * mul_prev + (long long)tok * mul_cur) % (long long)buckets;
  }
  const TW* w = table + (size_t)tok * hidden;
  const TW* b = pair + (size_t)r * hidden;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) o[i] = to_f32<TW>(w[i]) + to_f32<TW>(b[i]);
}

SI_EXPORT int si_embedding_pair(const int* tokens, const int* positions, const int* row_seq, const int* q_start,
                                const int* slots, int* last_token, const void* table, const void* pair,
                                int table_dtype, float* out, int num_tokens, int hidden, int vocab, int buckets,
                                long long mul_prev, long long mul_cur, int num_seqs, int* status,
                                cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (buckets <= 0 || mul_prev < 0 || mul_cur < 0) return -2;
  const int threads = hidden >= 1024 ? 256 : 128;
  if (table_dtype == SI_BF16)
    si_launch(embedding_pair_kernel<__nv_bfloat16>, dim3(num_tokens), dim3(threads), 0, stream, tokens, positions,
              row_seq, q_start, slots, last_token, (const __nv_bfloat16*)table, (const __nv_bfloat16*)pair, out,
              hidden, vocab, buckets, mul_prev, mul_cur, num_seqs, status);
  else
    si_launch(embedding_pair_kernel<float>, dim3(num_tokens), dim3(threads), 0, stream, tokens, positions, row_seq,
              q_start, slots, last_token, (const float*)table, (const float*)pair, out, hidden, vocab, buckets,
              mul_prev, mul_cur, num_seqs, status);
  return si_last_error();
}

// ---- a layer's own input for a token ------------------------------------------------------------------------------------
// out[t, j] = gelu_tanh(z[t, j]) * table[tokens[t] * stride + j] for j < dim, 0 for the columns from there to `width`; the table's
// slice of the layer starts at `table`. z and out in the compute dtype, as the table.
template <typename T>
__global__ void __launch_bounds__(256) token_gate_kernel(const T* __restrict__ z, long long z_stride, const int* __restrict__ tokens,
    const T* __restrict__ table, long long stride, T* __restrict__ out, long long out_stride, long long n, int width, int dim, int rows) {
  pdl_prologue();
  for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < n; idx += (long long)gridDim.x * blockDim.x) {
    const long long t = idx / width;
    const int j = (int)(idx - t * width), tok = tokens[t];
    float g = 0.f;
    if (j < dim && tok >= 0 && tok < rows) {
      const float v = to_f32<T>(z[t * z_stride + j]);
      g = 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v))) * to_f32<T>(table[(size_t)tok * stride + j]);
    }
    out[t * out_stride + j] = from_f32<T>(g);
  }
}

SI_EXPORT int si_token_gate(const void* z, int dtype, long long z_stride, const int* tokens, const void* table, long long stride,
                            void* out, long long out_stride, int num_tokens, int width, int dim, int rows, cudaStream_t stream) {
  if (num_tokens <= 0 || width <= 0) return 0;
  if (dim < 0 || dim > width) return -2;
  const long long n = (long long)num_tokens * width, want = (n + 255) / 256;
  const dim3 grid((unsigned)(want < 8LL * si_sm_count() ? want : 8LL * si_sm_count())), block(256);
  if (dtype == SI_BF16)
    si_launch(token_gate_kernel<__nv_bfloat16>, grid, block, 0, stream, (const __nv_bfloat16*)z, z_stride, tokens,
              (const __nv_bfloat16*)table, stride, (__nv_bfloat16*)out, out_stride, n, width, dim, rows);
  else
    si_launch(token_gate_kernel<float>, grid, block, 0, stream, (const float*)z, z_stride, tokens, (const float*)table, stride,
              (float*)out, out_stride, n, width, dim, rows);
  return si_last_error();
}
