// Layer norm with weight and (if there is one) bias over float32 rows:
//   y = (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * w + b,
// the mean first and the variance from the deviations, both float32 sums in a fixed order. One
// CTA per row; a thread keeps its PER elements of the row in registers between the passes.
//
// lrm_layer_norm: rows of the residual stream (all, or those `rows` names) -> activations. `partials`:
// float32 [n, T, h] slices of a product that are first added, in slice order, into the row, which is
// written back (a gathered row is not).
// lrm_layer_norm_conv: the same for a step of one token per sequence, and in the same pass the
// causal convolution over time in front of a mixer: h + sum_j taps[j] * (the h of n - 1 - j tokens
// ago), with the older rows from the sequence's tail [n - 1, h], which is moved on by one row.
// lrm_input_conv: that convolution alone, for steps of any number of tokens per sequence.
// lrm_layer_norm_add: a norm behind a sublayer, stream[t] += mult * y(sublayer output[t]), in
// place; with `cast_out` the updated row is also written in the activation type, which is what the
// next sublayer reads when nothing stands between it and the stream.
//
// Only the weight and the bias are `const __restrict__`: a load through such a pointer counts as
// invariant for the whole kernel and may be moved ahead of griddepcontrol.wait, next to the loads
// of w and b that stand there on purpose. What the kernel before this one writes (x, y, the stream)
// is read through plain pointers, whose loads stay behind the wait.
#include "common.cuh"

namespace {

template <int PER>
__device__ __forceinline__ void row_statistics(const float (&v)[PER], int hidden, float eps, float* scratch,
                                               float* mean_out, float* inv_out) {
  float sum = 0.f;
#pragma unroll
  for (int e = 0; e < PER; ++e) sum += v[e];  // elements beyond the row are zero
  const float mean = block_sum(sum, scratch) / static_cast<float>(hidden);
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int i = threadIdx.x + e * blockDim.x;
    const float dev = i < hidden ? v[e] - mean : 0.f;
    ss = fmaf(dev, dev, ss);
  }
  *mean_out = mean;
  *inv_out = 1.0f / sqrtf(block_sum(ss, scratch) / static_cast<float>(hidden) + eps);
}

// The row's elements, with the slices of a product that belong to it added in slice order.
template <int PER>
__device__ __forceinline__ void load_row(float (&v)[PER], float* x, size_t src, int hidden, const float* partials,
                                         int n_partials, size_t stride, bool write_back) {
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int i = threadIdx.x + e * blockDim.x;
    v[e] = i < hidden ? x[src + i] : 0.f;
  }
  if (n_partials <= 0) return;
  constexpr int kBatch = PER <= 8 ? 8 : 1;  // slices whose loads are in flight together
#pragma unroll 1
  for (int p0 = 0; p0 < n_partials; p0 += kBatch) {
#pragma unroll
    for (int e = 0; e < PER; ++e) {
      const int i = threadIdx.x + e * blockDim.x;
      float part[kBatch];
#pragma unroll
      for (int u = 0; u < kBatch; ++u)
        part[u] = i < hidden && p0 + u < n_partials ? partials[(p0 + u) * stride + src + i] : 0.f;
#pragma unroll
      for (int u = 0; u < kBatch; ++u)
        if (p0 + u < n_partials) v[e] += part[u];
    }
  }
  if (!write_back) return;
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int i = threadIdx.x + e * blockDim.x;
    if (i < hidden) x[src + i] = v[e];
  }
}

// Rows of up to 8 elements per thread take weight and bias into registers ahead of the wait;
// longer rows (PER 32, up to 1024 threads) read them where they are used, which keeps the kernel
// within the registers 1024 threads can have.
template <typename O, int PER>
__global__ __launch_bounds__(1024) void layer_norm_kernel(float* x, const float* __restrict__ w, const float* __restrict__ b, O* out,
                                  const int* rows, const float* partials, int n_partials, size_t partial_stride,
                                  int hidden, float eps) {
  __shared__ float scratch[32];
  constexpr bool EARLY = PER <= 8;
  constexpr int KEPT = EARLY ? PER : 1;
  float wv[KEPT], bv[KEPT];
  if (EARLY) {
#pragma unroll
    for (int e = 0; e < KEPT; ++e) {  // weights do not depend on the kernel before this one
      const int i = threadIdx.x + e * blockDim.x;
      wv[e] = i < hidden ? w[i] : 0.f;
      bv[e] = (b != nullptr && i < hidden) ? b[i] : 0.f;
    }
  }
  pdl_trigger();
  pdl_wait();
  const size_t src = static_cast<size_t>(rows != nullptr ? rows[blockIdx.x] : blockIdx.x) * hidden;
  float v[PER];
  load_row<PER>(v, x, src, hidden, partials, n_partials, partial_stride, rows == nullptr);
  float mean, inv;
  row_statistics<PER>(v, hidden, eps, scratch, &mean, &inv);
  const size_t dst = static_cast<size_t>(blockIdx.x) * hidden;
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int i = threadIdx.x + e * blockDim.x;
    if (i < hidden)
      out[dst + i] = from_f32<O>(fmaf((v[e] - mean) * inv, EARLY ? wv[e % KEPT] : w[i],
                                   EARLY ? bv[e % KEPT] : b != nullptr ? b[i] : 0.f));
  }
}

// One CTA per sequence, which brings one token: row b is sequence b's. A thread owns its channels, so
// it reads the tail's entries of a channel and moves them on without meeting anyone. The normalized
// row is rounded to the activation type before the convolution, as where the two are separate.
template <typename O, int PER>
__global__ __launch_bounds__(1024) void layer_norm_conv_kernel(float* x, const float* __restrict__ w,
                                       const float* __restrict__ b, O* out, const float* partials, int n_partials,
                                       size_t partial_stride, const float* __restrict__ taps, int n, float* tails,
                                       const int* __restrict__ slots, int hidden, float eps) {
  __shared__ float scratch[32];
  pdl_trigger();
  const int slot = slots[blockIdx.x];
  pdl_wait();
  const size_t src = static_cast<size_t>(blockIdx.x) * hidden;
  float v[PER];
  load_row<PER>(v, x, src, hidden, partials, n_partials, partial_stride, true);
  float mean, inv;
  row_statistics<PER>(v, hidden, eps, scratch, &mean, &inv);
  float* tail = slot >= 0 ? tails + static_cast<size_t>(slot) * (n - 1) * hidden : nullptr;
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int i = threadIdx.x + e * blockDim.x;
    if (i >= hidden) continue;
    const float h = to_f32(from_f32<O>(fmaf((v[e] - mean) * inv, w[i], b != nullptr ? b[i] : 0.f)));
    float acc = 0.f;
    if (tail != nullptr) {
      for (int s = 0; s < n - 1; ++s) {  // oldest first; entry s becomes what entry s + 1 was
        const float old = tail[static_cast<size_t>(s) * hidden + i];
        acc = fmaf(taps[static_cast<size_t>(s) * hidden + i], old, acc);
        if (s > 0) tail[static_cast<size_t>(s - 1) * hidden + i] = old;
      }
      tail[static_cast<size_t>(n - 2) * hidden + i] = h;
    }
    acc = fmaf(taps[static_cast<size_t>(n - 1) * hidden + i], h, acc);
    out[src + i] = from_f32<O>(h + acc);
  }
}

// out[t, c] = h[t, c] + sum_j taps[j, c] h[t - (n - 1) + j, c], the rows before a sequence's first token
// of the step from its tail [n - 1, width] (zeros at its start; a sequence of padding has zeros).
// The thread that finds a sequence's first token takes that sequence's first n - 1 tokens of the step
// together (the only ones that read the tail) and then writes the channel's new tail, the newest n - 1
// rows it has seen; the other threads leave those tokens out. So no entry is read after it is rewritten.
template <typename A>
__global__ void input_conv_kernel(const A* h, const float* __restrict__ taps, int n, float* tails, A* __restrict__ out,
                                  const int* __restrict__ cu_seqlens, const int* __restrict__ seq_of_token,
                                  const int* __restrict__ slots, int tokens, int per, int width) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= width) return;
  const int t0 = blockIdx.y * per, t1 = min(tokens, t0 + per);
  for (int t = t0; t < t1; ++t) {
    const int b = seq_of_token[t], start = cu_seqlens[b], local = t - start;
    if (local > 0 && local < n - 1) continue;
    if (local == 0 && n > 1) {
      const int slot = slots[b], m = cu_seqlens[b + 1] - start;
      float* tail = slot >= 0 ? tails + static_cast<size_t>(slot) * (n - 1) * width + c : nullptr;
      for (int l = 0; l < min(m, n - 1); ++l) {
        float acc = 0.f;
        for (int j = 0; j < n; ++j) {
          const int at = l - (n - 1) + j;  // the input's place among the step's tokens
          const float x = at >= 0 ? to_f32(h[static_cast<size_t>(start + at) * width + c])
                          : tail != nullptr ? tail[static_cast<size_t>(n - 1 + at) * width] : 0.f;
          acc = fmaf(taps[static_cast<size_t>(j) * width + c], x, acc);
        }
        const size_t o = static_cast<size_t>(start + l) * width + c;
        out[o] = from_f32<A>(to_f32(h[o]) + acc);
      }
      if (tail != nullptr)
        for (int s = 0; s < n - 1; ++s) {  // ascending: entry s + m lies above every entry written so far
          const int at = m - (n - 1) + s;
          tail[static_cast<size_t>(s) * width] = at >= 0 ? to_f32(h[static_cast<size_t>(start + at) * width + c])
                                                         : tail[static_cast<size_t>(s + m) * width];
        }
      continue;
    }
    float acc = 0.f;
    for (int j = 0; j < n; ++j)
      acc = fmaf(taps[static_cast<size_t>(j) * width + c], to_f32(h[static_cast<size_t>(t - (n - 1) + j) * width + c]), acc);
    const size_t o = static_cast<size_t>(t) * width + c;
    out[o] = from_f32<A>(to_f32(h[o]) + acc);
  }
}

template <typename O, int PER>
__global__ __launch_bounds__(1024) void layer_norm_add_kernel(float* stream, const float* y, const float* __restrict__ w,
                                      const float* __restrict__ b, float mult, O* cast_out, int hidden, float eps) {
  __shared__ float scratch[32];
  constexpr bool EARLY = PER <= 8;
  constexpr int KEPT = EARLY ? PER : 1;
  float wv[KEPT], bv[KEPT];
  if (EARLY) {
#pragma unroll
    for (int e = 0; e < KEPT; ++e) {
      const int i = threadIdx.x + e * blockDim.x;
      wv[e] = i < hidden ? w[i] : 0.f;
      bv[e] = (b != nullptr && i < hidden) ? b[i] : 0.f;
    }
  }
  pdl_trigger();
  pdl_wait();
  const size_t row = static_cast<size_t>(blockIdx.x) * hidden;
  float v[PER];
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int i = threadIdx.x + e * blockDim.x;
    v[e] = i < hidden ? y[row + i] : 0.f;
  }
  float mean, inv;
  row_statistics<PER>(v, hidden, eps, scratch, &mean, &inv);
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int i = threadIdx.x + e * blockDim.x;
    if (i < hidden) {
      const float updated = stream[row + i] + mult * fmaf((v[e] - mean) * inv, EARLY ? wv[e % KEPT] : w[i],
                                                          EARLY ? bv[e % KEPT] : b != nullptr ? b[i] : 0.f);
      stream[row + i] = updated;
      if (cast_out != nullptr) cast_out[row + i] = from_f32<O>(updated);
    }
  }
}

// short rows on 32 to 256 threads, rows beyond 2048 elements on 1024
int row_threads(int hidden) { return hidden > 2048 ? 1024 : (hidden >= 1024 ? 256 : (hidden >= 256 ? 128 : 32)); }

}  // namespace

// x float32 [*, hidden]; w float32 [hidden], b likewise or null; rows int32 [n_rows] or null (row r of
// out is row r of x); partials float32, n_partials planes partial_stride apart, or null.
LRM_API int lrm_layer_norm(float* x, const float* w, const float* b, void* out, int out_dtype, const int* rows,
                           int n_rows, int hidden, float eps, const float* partials, int n_partials,
                           long long partial_stride, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (hidden <= 0 || !(eps > 0.f) || x == nullptr || w == nullptr || out == nullptr ||
      n_partials < 0 || (n_partials > 0 && partials == nullptr))
    return LRM_BAD_ARGUMENT;
  const int threads = row_threads(hidden), per = (hidden + threads - 1) / threads;
#define LRM_LAYER_NORM(OT, PER)                                                                                   \
  do {                                                                                                            \
    LRM_LAUNCH((layer_norm_kernel<OT, PER>), n_rows, threads, 0, stream, x, w, b, static_cast<OT*>(out), rows, \
               partials, n_partials, static_cast<size_t>(partial_stride), hidden, eps);                                                                                              \
    return 0;                                                                                                     \
  } while (0)
  if (out_dtype == LRM_F32) {
    if (per <= 4) LRM_LAYER_NORM(float, 4);
    if (per <= 8) LRM_LAYER_NORM(float, 8);
    if (per <= 32) LRM_LAYER_NORM(float, 32);
  } else if (out_dtype == LRM_BF16) {
    if (per <= 4) LRM_LAYER_NORM(__nv_bfloat16, 4);
    if (per <= 8) LRM_LAYER_NORM(__nv_bfloat16, 8);
    if (per <= 32) LRM_LAYER_NORM(__nv_bfloat16, 32);
  } else {
    return LRM_BAD_ARGUMENT;
  }
#undef LRM_LAYER_NORM
  return LRM_UNSUPPORTED;  // rows longer than 32768 elements
}

// stream, y float32 [n_rows, hidden]; cast_out [n_rows, hidden] in out_dtype, or null.
LRM_API int lrm_layer_norm_add(float* stream_rows, const float* y, const float* w, const float* b, float mult,
                               void* cast_out, int out_dtype, int n_rows, int hidden, float eps,
                               cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (hidden <= 0 || !(eps > 0.f) || stream_rows == nullptr || y == nullptr || w == nullptr)
    return LRM_BAD_ARGUMENT;
  const int threads = row_threads(hidden), per = (hidden + threads - 1) / threads;
#define LRM_LAYER_NORM_ADD(OT, PER)                                                                             \
  do {                                                                                                          \
    LRM_LAUNCH((layer_norm_add_kernel<OT, PER>), n_rows, threads, 0, stream, stream_rows, y, w, b, mult,        \
               static_cast<OT*>(cast_out), hidden, eps);                                                        \
    return 0;                                                                                                   \
  } while (0)
  if (out_dtype == LRM_F32) {
    if (per <= 4) LRM_LAYER_NORM_ADD(float, 4);
    if (per <= 8) LRM_LAYER_NORM_ADD(float, 8);
    if (per <= 32) LRM_LAYER_NORM_ADD(float, 32);
  } else if (out_dtype == LRM_BF16) {
    if (per <= 4) LRM_LAYER_NORM_ADD(__nv_bfloat16, 4);
    if (per <= 8) LRM_LAYER_NORM_ADD(__nv_bfloat16, 8);
    if (per <= 32) LRM_LAYER_NORM_ADD(__nv_bfloat16, 32);
  } else {
    return LRM_BAD_ARGUMENT;
  }
#undef LRM_LAYER_NORM_ADD
  return LRM_UNSUPPORTED;
}

// x float32 [seqs, hidden], row b the one token of sequence b; taps float32 [n, hidden] (the last row
// the current token's), n > 1; tails float32 [slots, n - 1, hidden]; the rest as for lrm_layer_norm.
LRM_API int lrm_layer_norm_conv(float* x, const float* w, const float* b, void* out, int out_dtype,
                                const float* partials, int n_partials, long long partial_stride, const float* taps,
                                int n, float* tails, const int* slots, int seqs, int hidden, float eps,
                                cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (hidden <= 0 || !(eps > 0.f) || x == nullptr || w == nullptr || out == nullptr || taps == nullptr || n <= 1 ||
      tails == nullptr || slots == nullptr || n_partials < 0 || (n_partials > 0 && partials == nullptr))
    return LRM_BAD_ARGUMENT;
  const int threads = row_threads(hidden), per = (hidden + threads - 1) / threads;
#define LRM_NORM_CONV(OT, PER)                                                                                    \
  do {                                                                                                            \
    LRM_LAUNCH((layer_norm_conv_kernel<OT, PER>), seqs, threads, 0, stream, x, w, b, static_cast<OT*>(out), partials, \
               n_partials, static_cast<size_t>(partial_stride), taps, n, tails, slots, hidden, eps);              \
    return 0;                                                                                                     \
  } while (0)
  if (out_dtype == LRM_F32) {
    if (per <= 4) LRM_NORM_CONV(float, 4);
    if (per <= 8) LRM_NORM_CONV(float, 8);
    if (per <= 32) LRM_NORM_CONV(float, 32);
  } else if (out_dtype == LRM_BF16) {
    if (per <= 4) LRM_NORM_CONV(__nv_bfloat16, 4);
    if (per <= 8) LRM_NORM_CONV(__nv_bfloat16, 8);
    if (per <= 32) LRM_NORM_CONV(__nv_bfloat16, 32);
  } else {
    return LRM_BAD_ARGUMENT;
  }
#undef LRM_NORM_CONV
  return LRM_UNSUPPORTED;
}

// h, out [tokens, width] of `dtype`; taps float32 [n, width]; tails float32 [slots, n - 1, width] (null
// when n is 1).
LRM_API int lrm_input_conv(const void* h, int dtype, const float* taps, int n, float* tails, void* out,
                           const int* cu_seqlens, const int* seq_of_token, const int* slots, int tokens, int width,
                           cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (width <= 0 || n <= 0 || taps == nullptr || (n > 1 && tails == nullptr)) return LRM_BAD_ARGUMENT;
  // a thread walks several consecutive tokens of its channel (their rows are read again from L1)
  const int threads = width >= 256 ? 256 : ((width + 31) / 32) * 32;
  const int columns = (width + threads - 1) / threads;
  int per = 1;
  while (per < 8 && static_cast<long long>(columns) * ((tokens + 2 * per - 1) / (2 * per)) >= 148 * 8) per *= 2;
  const int rows = (tokens + per - 1) / per;
  if (rows > 65535) return LRM_UNSUPPORTED;
  const dim3 grid(columns, rows);
  if (dtype == LRM_F32)
    LRM_LAUNCH(input_conv_kernel<float>, grid, threads, 0, stream, static_cast<const float*>(h), taps, n, tails,
               static_cast<float*>(out), cu_seqlens, seq_of_token, slots, tokens, per, width);
  else if (dtype == LRM_BF16)
    LRM_LAUNCH(input_conv_kernel<__nv_bfloat16>, grid, threads, 0, stream, static_cast<const __nv_bfloat16*>(h), taps,
               n, tails, static_cast<__nv_bfloat16*>(out), cu_seqlens, seq_of_token, slots, tokens, per, width);
  else
    return LRM_BAD_ARGUMENT;
  return 0;
}
