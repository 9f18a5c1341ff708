// Layer norm with weight and (if there is one) bias over float32 rows:
//   y = (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * w + b,
// the mean first and the variance from the deviations, both float32 sums in a fixed order. One
// CTA per row; a thread keeps its PER elements of the row in registers between the passes.
//
// lrm_layer_norm: rows of the residual stream (all, or those `rows` names) -> activations. `partials`:
// float32 [n, T, h] slices of a product that are first added, in slice order, into the row, which is
// written back (a gathered row is not); rows of up to 8192 elements. `add`: float32 [h], added to every row of the
// stream once the row that is normalized has been read (the bias of an output that joins the stream later).
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

// Where element e of a thread's PER elements stands in the row: VEC consecutive ones at a time.
template <int VEC>
__device__ __forceinline__ int element(int e) {
  return (threadIdx.x + (e / VEC) * blockDim.x) * VEC + e % VEC;
}

// Elements of a row of length `hidden` (a multiple of VEC), zero beyond it; VEC 4 with 16-byte accesses.
template <int PER, int VEC>
__device__ __forceinline__ void read_row(float (&v)[PER], const float* row, int hidden) {
#pragma unroll
  for (int e = 0; e < PER; e += VEC) {
    const int i = element<VEC>(e);
    if constexpr (VEC == 4) {
      const float4 x = i < hidden ? *reinterpret_cast<const float4*>(row + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      v[e] = x.x, v[e + 1] = x.y, v[e + 2] = x.z, v[e + 3] = x.w;
    } else {
      v[e] = i < hidden ? row[i] : 0.f;
    }
  }
}

template <int PER, int VEC, typename O>
__device__ __forceinline__ void write_row(const float (&v)[PER], O* row, int hidden) {
#pragma unroll
  for (int e = 0; e < PER; e += VEC) {
    const int i = element<VEC>(e);
    if (i >= hidden) continue;
    if constexpr (VEC == 4 && sizeof(O) == 4) {
      *reinterpret_cast<float4*>(row + i) = make_float4(v[e], v[e + 1], v[e + 2], v[e + 3]);
    } else if constexpr (VEC == 4) {
      __nv_bfloat162 lo = __floats2bfloat162_rn(v[e], v[e + 1]), hi = __floats2bfloat162_rn(v[e + 2], v[e + 3]);
      *reinterpret_cast<uint2*>(row + i) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
    } else {
      row[i] = from_f32<O>(v[e]);
    }
  }
}

// The row's elements, with the slices of a product that belong to it added in slice order.
template <int PER, int VEC>
__device__ __forceinline__ void load_row(float (&v)[PER], float* x, size_t src, int hidden, const float* partials,
                                         int n_partials, size_t stride, bool write_back) {
  read_row<PER, VEC>(v, x + src, hidden);
  if constexpr (PER <= 8) {  // longer rows have no registers to spare: the host adds their slices first
    if (n_partials <= 0) return;
#pragma unroll 1
    for (int p = 0; p < n_partials; p += 2) {  // two slices' loads are in flight together
      float first[PER], second[PER];
      read_row<PER, VEC>(first, partials + p * stride + src, hidden);
      if (p + 1 < n_partials) read_row<PER, VEC>(second, partials + (p + 1) * stride + src, hidden);
#pragma unroll
      for (int e = 0; e < PER; ++e) {
        v[e] += first[e];
        if (p + 1 < n_partials) v[e] += second[e];
      }
    }
    if (write_back) write_row<PER, VEC>(v, x + src, hidden);
  }
}

template <int PER, int VEC>
__device__ __forceinline__ void normalize(float (&v)[PER], int hidden, float eps, float* scratch) {
  float sum = 0.f;
#pragma unroll
  for (int e = 0; e < PER; ++e) sum += v[e];  // elements beyond the row are zero
  const float mean = block_sum(sum, scratch) / static_cast<float>(hidden);
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    v[e] = element<VEC>(e) < hidden ? v[e] - mean : 0.f;
    ss = fmaf(v[e], v[e], ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / static_cast<float>(hidden) + eps);
#pragma unroll
  for (int e = 0; e < PER; ++e) v[e] *= inv;
}

// Rows of up to 8 elements per thread take weight and bias into registers ahead of the wait;
// longer rows (PER 32, up to 1024 threads) read them where they are used, which keeps the kernel
// within the registers 1024 threads can have.
template <typename O, int PER, int VEC>
__global__ __launch_bounds__(1024) void layer_norm_kernel(float* x, const float* __restrict__ w, const float* __restrict__ b, O* out,
                                  const int* rows, const float* partials, int n_partials, size_t partial_stride,
                                  const float* __restrict__ add, int hidden, float eps) {
  __shared__ float scratch[32];
  constexpr bool EARLY = PER <= 8;
  constexpr int KEPT = EARLY ? PER : VEC;
  float wv[KEPT], bv[KEPT] = {};
  if constexpr (EARLY) {  // weights do not depend on the kernel before this one
    read_row<KEPT, VEC>(wv, w, hidden);
    if (b != nullptr) read_row<KEPT, VEC>(bv, b, hidden);
  }
  pdl_trigger();
  pdl_wait();
  const size_t src = static_cast<size_t>(rows != nullptr ? rows[blockIdx.x] : blockIdx.x) * hidden;
  float v[PER];
  load_row<PER, VEC>(v, x, src, hidden, partials, n_partials, partial_stride, rows == nullptr && add == nullptr);
  if constexpr (EARLY) {
    if (add != nullptr) {
      float moved[PER];
      read_row<PER, VEC>(moved, add, hidden);
#pragma unroll
      for (int e = 0; e < PER; ++e) moved[e] += v[e];
      write_row<PER, VEC>(moved, x + src, hidden);
    }
  }
  normalize<PER, VEC>(v, hidden, eps, scratch);
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int i = element<VEC>(e);
    if (i < hidden) v[e] = fmaf(v[e], EARLY ? wv[e % KEPT] : w[i], EARLY ? bv[e % KEPT] : b != nullptr ? b[i] : 0.f);
  }
  write_row<PER, VEC>(v, out + static_cast<size_t>(blockIdx.x) * hidden, hidden);
}

// One CTA per sequence, which brings one token: row b is sequence b's. A thread owns its channels, so
// it reads the tail's entries of a channel and moves them on without meeting anyone. The normalized
// row is rounded to the activation type before the convolution, as where the two are separate.
template <typename O, int PER, int VEC>
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
  load_row<PER, VEC>(v, x, src, hidden, partials, n_partials, partial_stride, true);
  normalize<PER, VEC>(v, hidden, eps, scratch);
  float* tail = slot >= 0 ? tails + static_cast<size_t>(slot) * (n - 1) * hidden : nullptr;
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int i = element<VEC>(e);
    if (i < hidden) v[e] = to_f32(from_f32<O>(fmaf(v[e], w[i], b != nullptr ? b[i] : 0.f)));
  }
  float y[PER], tap[PER], old[PER];
  read_row<PER, VEC>(tap, taps + static_cast<size_t>(n - 1) * hidden, hidden);
#pragma unroll
  for (int e = 0; e < PER; ++e) y[e] = 0.f;
  if (tail != nullptr) {
#pragma unroll 1
    for (int s = 0; s < n - 1; ++s) {  // oldest first; entry s becomes what entry s + 1 was
      float older[PER];
      read_row<PER, VEC>(old, tail + static_cast<size_t>(s) * hidden, hidden);
      read_row<PER, VEC>(older, taps + static_cast<size_t>(s) * hidden, hidden);
#pragma unroll
      for (int e = 0; e < PER; ++e) y[e] = fmaf(older[e], old[e], y[e]);
      if (s > 0) write_row<PER, VEC>(old, tail + static_cast<size_t>(s - 1) * hidden, hidden);
    }
    write_row<PER, VEC>(v, tail + static_cast<size_t>(n - 2) * hidden, hidden);
  }
#pragma unroll
  for (int e = 0; e < PER; ++e) y[e] = v[e] + fmaf(tap[e], v[e], y[e]);
  write_row<PER, VEC>(y, out + src, hidden);
}

// out[t, c] = h[t, c] + sum_j taps[j, c] h[t - (n - 1) + j, c], the rows before a sequence's first token
// of the step from its tail [n - 1, width] (zeros at its start; a sequence of padding has zeros).
// The thread that finds a sequence's first token takes that sequence's first n - 1 tokens of the step
// together (the only ones that read the tail) and then writes the channel's new tail, the newest n - 1
// rows it has seen; the other threads leave those tokens out. So no entry is read after it is rewritten.
// N: the taps, when they are few (a thread then keeps the last N rows of its channels in registers), or 0.
// VEC channels per thread.
template <typename A, int N, int VEC>
__global__ void input_conv_kernel(const A* h, const float* __restrict__ taps, int n_any, float* tails,
                                  A* __restrict__ out, const int* __restrict__ cu_seqlens,
                                  const int* __restrict__ seq_of_token, const int* __restrict__ slots, int tokens,
                                  int per, int width) {
  pdl_trigger();
  const int n = N > 0 ? N : n_any;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  const int t0 = blockIdx.y * per, t1 = min(tokens, t0 + per);
  if (c >= width || t0 >= t1) return;
  int b = seq_of_token[t0], start = cu_seqlens[b], end = cu_seqlens[b + 1];
  float tap[N > 0 ? N : 1][VEC];
  if constexpr (N > 0) {
#pragma unroll
    for (int j = 0; j < N; ++j)
#pragma unroll
      for (int e = 0; e < VEC; ++e) tap[j][e] = taps[static_cast<size_t>(j) * width + c + e];
  }
  pdl_wait();
  auto load = [&](int t, float (&x)[VEC]) {
    const A* src = h + static_cast<size_t>(t) * width + c;
    if constexpr (VEC == 2 && sizeof(A) == 2) {
      const uint32_t raw = *reinterpret_cast<const uint32_t*>(src);
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw));
      x[0] = f.x, x[1] = f.y;
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] = to_f32(src[e]);
    }
  };
  auto store = [&](int t, const float (&y)[VEC]) {
    A* dst = out + static_cast<size_t>(t) * width + c;
    if constexpr (VEC == 2 && sizeof(A) == 2) {
      __nv_bfloat162 v = __floats2bfloat162_rn(y[0], y[1]);
      *reinterpret_cast<uint32_t*>(dst) = *reinterpret_cast<uint32_t*>(&v);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) dst[e] = from_f32<A>(y[e]);
    }
  };
  float window[N > 1 ? N - 1 : 1][VEC];  // rows t - (N - 1) .. t - 1
  bool kept = false;                       // the window holds them
  for (int t = t0; t < t1; ++t) {
    while (t >= end) {
      start = end;
      end = cu_seqlens[++b + 1];
    }
    const int local = t - start;
    if (local < n - 1) {
      kept = false;
      if (local > 0) continue;
      const int slot = slots[b], m = end - start;
      float* tail = slot >= 0 ? tails + static_cast<size_t>(slot) * (n - 1) * width + c : nullptr;
      for (int l = 0; l < min(m, n - 1); ++l) {
        float acc[VEC] = {}, x[VEC];
        for (int j = 0; j < n; ++j) {
          const int at = l - (n - 1) + j;  // the input's place among the step's tokens
          if (at >= 0) load(start + at, x);
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            if (at < 0) x[e] = tail != nullptr ? tail[static_cast<size_t>(n - 1 + at) * width + e] : 0.f;
            acc[e] = fmaf(taps[static_cast<size_t>(j) * width + c + e], x[e], acc[e]);
          }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] += x[e];  // the last input read is the token's own
        store(start + l, acc);
      }
      if (tail != nullptr)
        for (int s = 0; s < n - 1; ++s) {  // ascending: entry s + m lies above every entry written so far
          const int at = m - (n - 1) + s;
          float x[VEC];
          if (at >= 0) load(start + at, x);
#pragma unroll
          for (int e = 0; e < VEC; ++e)
            tail[static_cast<size_t>(s) * width + e] = at >= 0 ? x[e] : tail[static_cast<size_t>(s + m) * width + e];
        }
      continue;
    }
    float acc[VEC] = {}, x[VEC];
    if constexpr (N > 0) {
      if (!kept) {
#pragma unroll
        for (int j = 0; j < N - 1; ++j) load(t - (N - 1) + j, window[j]);
        kept = true;
      }
      load(t, x);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
#pragma unroll
        for (int j = 0; j < N - 1; ++j) acc[e] = fmaf(tap[j][e], window[j][e], acc[e]);
        acc[e] = fmaf(tap[N - 1][e], x[e], acc[e]) + x[e];
#pragma unroll
        for (int j = 0; j + 1 < N - 1; ++j) window[j][e] = window[j + 1][e];
        if (N > 1) window[N > 1 ? N - 2 : 0][e] = x[e];
      }
    } else {
      for (int j = 0; j < n; ++j) {
        load(t - (n - 1) + j, x);
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = fmaf(taps[static_cast<size_t>(j) * width + c + e], x[e], acc[e]);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] += x[e];
    }
    store(t, acc);
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

// 16-byte accesses: rows of whole groups of four that begin on 16-byte boundaries
bool fours(int hidden, long long partial_stride, const void* x, const void* w, const void* b, const void* out,
           const void* partials) {
  const uintptr_t all = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(b) |
                        reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(partials);
  return hidden % 4 == 0 && partial_stride % 4 == 0 && all % 16 == 0;
}

}  // namespace

// x float32 [*, hidden]; w float32 [hidden], b likewise or null; rows int32 [n_rows] or null (row r of
// out is row r of x); partials float32, n_partials planes partial_stride apart, or null; add float32
// [hidden] or null (not with rows).
LRM_API int lrm_layer_norm(float* x, const float* w, const float* b, void* out, int out_dtype, const int* rows,
                           int n_rows, int hidden, float eps, const float* partials, int n_partials,
                           long long partial_stride, const float* add, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (hidden <= 0 || !(eps > 0.f) || x == nullptr || w == nullptr || out == nullptr ||
      n_partials < 0 || (n_partials > 0 && partials == nullptr) || (add != nullptr && rows != nullptr))
    return LRM_BAD_ARGUMENT;
  const int threads = row_threads(hidden), per = (hidden + threads - 1) / threads;
  if (per > 8 && (n_partials > 0 || add != nullptr)) return LRM_UNSUPPORTED;
  const bool four = fours(hidden, partial_stride, x, w, b, out, partials) && reinterpret_cast<uintptr_t>(add) % 16 == 0;
#define LRM_LAYER_NORM(OT, PER)                                                                                   \
  do {                                                                                                            \
    if (four)                                                                                                     \
      LRM_LAUNCH((layer_norm_kernel<OT, PER, 4>), n_rows, threads, 0, stream, x, w, b, static_cast<OT*>(out), rows, \
                 partials, n_partials, static_cast<size_t>(partial_stride), add, hidden, eps);                    \
    else                                                                                                          \
      LRM_LAUNCH((layer_norm_kernel<OT, PER, 1>), n_rows, threads, 0, stream, x, w, b, static_cast<OT*>(out), rows, \
                 partials, n_partials, static_cast<size_t>(partial_stride), add, hidden, eps);                    \
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
// the current token's), n > 1; tails float32 [slots, n - 1, hidden]; rows of up to 8192 elements; the rest as
// for lrm_layer_norm.
LRM_API int lrm_layer_norm_conv(float* x, const float* w, const float* b, void* out, int out_dtype,
                                const float* partials, int n_partials, long long partial_stride, const float* taps,
                                int n, float* tails, const int* slots, int seqs, int hidden, float eps,
                                cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (hidden <= 0 || !(eps > 0.f) || x == nullptr || w == nullptr || out == nullptr || taps == nullptr || n <= 1 ||
      tails == nullptr || slots == nullptr || n_partials < 0 || (n_partials > 0 && partials == nullptr))
    return LRM_BAD_ARGUMENT;
  const int threads = row_threads(hidden), per = (hidden + threads - 1) / threads;
  const bool four = fours(hidden, partial_stride, x, w, b, out, partials) &&
                    (reinterpret_cast<uintptr_t>(taps) | reinterpret_cast<uintptr_t>(tails)) % 16 == 0;
#define LRM_NORM_CONV(OT, PER)                                                                                    \
  do {                                                                                                            \
    if (four)                                                                                                     \
      LRM_LAUNCH((layer_norm_conv_kernel<OT, PER, 4>), seqs, threads, 0, stream, x, w, b, static_cast<OT*>(out),    \
                 partials, n_partials, static_cast<size_t>(partial_stride), taps, n, tails, slots, hidden, eps);  \
    else                                                                                                          \
      LRM_LAUNCH((layer_norm_conv_kernel<OT, PER, 1>), seqs, threads, 0, stream, x, w, b, static_cast<OT*>(out),    \
                 partials, n_partials, static_cast<size_t>(partial_stride), taps, n, tails, slots, hidden, eps);  \
    return 0;                                                                                                     \
  } while (0)
  if (out_dtype == LRM_F32) {
    if (per <= 4) LRM_NORM_CONV(float, 4);
    if (per <= 8) LRM_NORM_CONV(float, 8);
  } else if (out_dtype == LRM_BF16) {
    if (per <= 4) LRM_NORM_CONV(__nv_bfloat16, 4);
    if (per <= 8) LRM_NORM_CONV(__nv_bfloat16, 8);
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
  const bool two = width % 2 == 0 && (reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(out)) % 8 == 0;
  // a thread walks several consecutive tokens of its channels (the rows it has read stay in registers)
  const int groups = two ? width / 2 : width;
  const int threads = groups >= 256 ? 256 : ((groups + 31) / 32) * 32;
  const int columns = (groups + threads - 1) / threads;
  int per = 1;
  while (per < 16 && static_cast<long long>(columns) * ((tokens + 2 * per - 1) / (2 * per)) >= 148 * 6) per *= 2;
  const int rows = (tokens + per - 1) / per;
  if (rows > 65535) return LRM_UNSUPPORTED;
  const dim3 grid(columns, rows);
#define LRM_CONV_N(AT, V, TAPS)                                                                                  \
  LRM_LAUNCH((input_conv_kernel<AT, TAPS, V>), grid, threads, 0, stream, static_cast<const AT*>(h), taps, n, tails, \
             static_cast<AT*>(out), cu_seqlens, seq_of_token, slots, tokens, per, width)
#define LRM_CONV(AT, V)                                \
  do {                                                 \
    if (n == 2) LRM_CONV_N(AT, V, 2);                  \
    else if (n == 3) LRM_CONV_N(AT, V, 3);             \
    else if (n == 4) LRM_CONV_N(AT, V, 4);             \
    else LRM_CONV_N(AT, V, 0);                         \
  } while (0)
  if (dtype == LRM_F32) {
    if (two) LRM_CONV(float, 2); else LRM_CONV(float, 1);
  } else if (dtype == LRM_BF16) {
    if (two) LRM_CONV(__nv_bfloat16, 2); else LRM_CONV(__nv_bfloat16, 1);
  } else {
    return LRM_BAD_ARGUMENT;
  }
#undef LRM_CONV
#undef LRM_CONV_N
  return 0;
}
