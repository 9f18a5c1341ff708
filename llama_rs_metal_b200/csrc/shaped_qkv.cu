// The split of a step's fused q|k|v projection for attention layers that shape their queries and
// keys on the way: one CTA per token takes the projection row [q_heads * d | kv_heads * d |
// kv_heads * dv] (rows may be further apart than that: columns behind it belong to someone else)
// through, in this order and each only if asked for,
//   1. the projections' biases (float32 [row]);
//   2. a short causal convolution over time per channel (taps [n, row], the last row the current
//      token's, no bias, zeros before the sequence's start); inputs before the step's first token
//      come from the sequence's tail [n - 1, row] of unbiased projections in the state storage,
//      the bias added here where the input's position is not before the start;
//   3. an RMS norm over the whole query part and one over the whole key part, with weights;
//   4. an RMS norm over every query head and every key head, with one weight of size d for all
//      query heads and one for all key heads;
//   5. a rotation by position of the first `rotary` dimensions of every query and key head,
//      dimension i paired with i + rotary/2 (pairing 0) or 2i with 2i + 1 (pairing 1), angle =
//      position * inv_freq[i] formed in double precision, here or, for layers that share their
//      frequencies, once per step in a table of cosines and sines (lrm_rope_table64); `magnitude`
//      multiplies cosines and sines (a table holds it already);
//   6. the division of every query and key head by its root mean square (no weight),
// and writes q, k, v in the activation type: q packed, k and v packed (when asked for) and into
// the paged cache at dest_rows[t] (see qkv_store.cu for the layout). Everything between the
// projection and the rounding at the end is float32. Reads of the projection go through plain
// pointers: it is the output of the kernel before.
//
// Layers with biases and a split-half rotation at most (steps 1 and 5, from a table) take four columns per
// thread, all loads and stores 16 or 8 bytes wide, wherever sizes and addresses allow (split_rotate_kernel).
// Layers without a convolution, a row norm and a division behind the rotation (steps 1, 4 and 5 at
// most) otherwise run a kernel of their own: a warp takes a head from its projection to its stores in registers,
// with no barrier after the table of cosines and sines.
#include "common.cuh"

namespace {

template <typename S, typename A>
__global__ void shaped_qkv_kernel(const S* proj, long long stride, const float* __restrict__ bias, const float* __restrict__ taps, int n,
                                  const float* tails, const int* __restrict__ cu_seqlens,
                                  const int* __restrict__ seq_of_token, const int* __restrict__ slots,
                                  const int* __restrict__ positions, const float* __restrict__ q_norm,
                                  const float* __restrict__ k_norm, float row_eps,
                                  const float* __restrict__ q_head_w, const float* __restrict__ k_head_w,
                                  float head_w_eps, const double* __restrict__ inv_freq, double magnitude, const float2* table,
                                  int rotary, int pairing, int head_norm,
                                  float head_eps, A* __restrict__ q_out, A* __restrict__ k_out,
                                  A* __restrict__ v_out, A* __restrict__ k_pages, A* __restrict__ v_pages,
                                  const int* __restrict__ dest_rows, int q_heads, int kv_heads, int d, int dv,
                                  int page_size) {
  extern __shared__ float smem[];
  __shared__ float scratch[32];
  const int nq = q_heads * d, nk = kv_heads * d, nv = kv_heads * dv;
  const int width = nq + nk + nv, half = rotary / 2;
  float* row = smem;            // [width]
  float* cs = smem + width;     // [half] cosines, then [half] sines
  pdl_trigger();
  const int t = blockIdx.x;
  const int pos = positions[t];
  if (table == nullptr)
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
      double sn, c;
      sincos(static_cast<double>(pos) * inv_freq[i], &sn, &c);
      cs[i] = static_cast<float>(c * magnitude);
      cs[half + i] = static_cast<float>(sn * magnitude);
    }
  pdl_wait();
  if (table != nullptr)
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
      const float2 entry = table[static_cast<size_t>(t) * half + i];
      cs[i] = entry.x;
      cs[half + i] = entry.y;
    }
  const S* src = proj + static_cast<size_t>(t) * stride;
  if (taps == nullptr || n <= 1) {
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
      float x = to_f32(src[c]) + (bias != nullptr ? bias[c] : 0.f);
      if (taps != nullptr) x *= taps[c];
      row[c] = x;
    }
  } else {
    const int b = seq_of_token[t], local = t - cu_seqlens[b], slot = slots[b];
    const float* tail = slot >= 0 ? tails + static_cast<size_t>(slot) * (n - 1) * width : nullptr;
    // a thread takes kGroup columns at a time, so that the loads of one input row are all under way
    // before the first is used (one column after another, a CTA waited for n loads in turn per column)
    constexpr int kGroup = 8;
    for (int first = 0; first < width; first += kGroup * blockDim.x) {
      float acc[kGroup], add[kGroup];
#pragma unroll
      for (int e = 0; e < kGroup; ++e) {
        const int c = first + e * blockDim.x + threadIdx.x;
        acc[e] = 0.f;
        add[e] = (bias != nullptr && c < width) ? bias[c] : 0.f;
      }
      for (int back = n - 1; back >= 0; --back) {  // oldest input first
        if (pos - back < 0) continue;              // before the sequence's start: zero
        const int at = local - back;
        const S* from_step = at >= 0 ? proj + static_cast<size_t>(t - back) * stride : nullptr;
        const float* from_tail = (at < 0 && tail != nullptr) ? tail + static_cast<size_t>(n - 1 + at) * width : nullptr;
        const float* tap = taps + static_cast<size_t>(n - 1 - back) * width;
#pragma unroll
        for (int e = 0; e < kGroup; ++e) {
          const int c = first + e * blockDim.x + threadIdx.x;
          if (c < width) {
            const float x = from_step != nullptr ? to_f32(from_step[c]) : from_tail != nullptr ? from_tail[c] : 0.f;
            acc[e] = fmaf(tap[c], x + add[e], acc[e]);
          }
        }
      }
#pragma unroll
      for (int e = 0; e < kGroup; ++e) {
        const int c = first + e * blockDim.x + threadIdx.x;
        if (c < width) row[c] = acc[e];
      }
    }
  }
  __syncthreads();
  if (q_norm != nullptr) {
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x; c < nq + nk; c += blockDim.x) {
      const float x = row[c];
      if (c < nq) sq = fmaf(x, x, sq); else sk = fmaf(x, x, sk);
    }
    const float inv_q = 1.0f / sqrtf(block_sum(sq, scratch) / static_cast<float>(nq) + row_eps);
    const float total_k = block_sum(sk, scratch);
    const float inv_k = nk > 0 ? 1.0f / sqrtf(total_k / static_cast<float>(nk) + row_eps) : 0.f;
    for (int c = threadIdx.x; c < nq + nk; c += blockDim.x)
      row[c] = c < nq ? row[c] * inv_q * q_norm[c] : row[c] * inv_k * k_norm[c - nq];
    __syncthreads();
  }
  if (q_head_w != nullptr) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    for (int hd = warp; hd < q_heads + kv_heads; hd += warps) {
      float* head = row + hd * d;
      const float* w = hd < q_heads ? q_head_w : k_head_w;
      float ss = 0.f;
      for (int i = lane; i < d; i += 32) ss = fmaf(head[i], head[i], ss);
      const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(d) + head_w_eps);
      for (int i = lane; i < d; i += 32) head[i] = (head[i] * inv) * w[i];
    }
    __syncthreads();
  }
  if (half > 0) {
    const int heads = q_heads + kv_heads;  // query heads, then key heads, are contiguous rows of d
    for (int idx = threadIdx.x; idx < heads * half; idx += blockDim.x) {
      const int hd = idx / half, i = idx % half;
      float* head = row + hd * d;
      const int a = pairing == 0 ? i : 2 * i, b2 = pairing == 0 ? i + half : 2 * i + 1;
      const float u = head[a], v = head[b2], c = cs[i], sn = cs[half + i];
      head[a] = fmaf(u, c, -__fmul_rn(v, sn));
      head[b2] = fmaf(v, c, __fmul_rn(u, sn));
    }
    __syncthreads();
  }
  if (head_norm) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    for (int hd = warp; hd < q_heads + kv_heads; hd += warps) {
      float* head = row + hd * d;
      float ss = 0.f;
      for (int i = lane; i < d; i += 32) ss = fmaf(head[i], head[i], ss);
      const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(d) + head_eps);
      for (int i = lane; i < d; i += 32) head[i] *= inv;
    }
    __syncthreads();
  }
  const int dest = k_pages != nullptr ? dest_rows[t] : -1;
  const long long page = dest >= 0 ? dest / page_size : -1;
  const int in_page = dest >= 0 ? dest % page_size : 0;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const A val = from_f32<A>(row[c]);
    if (c < nq) {
      q_out[static_cast<size_t>(t) * nq + c] = val;
    } else if (c < nq + nk) {
      const int e = c - nq, kh = e / d, j = e % d;
      if (k_out != nullptr) k_out[static_cast<size_t>(t) * nk + e] = val;
      if (page >= 0) k_pages[((static_cast<size_t>(page) * kv_heads + kh) * page_size + in_page) * d + j] = val;
    } else {
      const int e = c - nq - nk, kh = e / dv, j = e % dv;
      if (v_out != nullptr) v_out[static_cast<size_t>(t) * nv + e] = val;
      if (page >= 0) v_pages[((static_cast<size_t>(page) * kv_heads + kh) * page_size + in_page) * dv + j] = val;
    }
  }
}

// gridDim.y CTAs per token share its heads, one warp per head at a time; lane l holds elements VEC l .. of every group of
// 32 VEC (VEC 2 where d, dv, the row pitch and all addresses allow pairs).
constexpr int kHeadPer = 8;  // elements of a head one lane holds at most: heads of up to 256

template <typename S, typename A, int VEC>
__global__ void shaped_heads_kernel(const S* proj, long long stride, const float* __restrict__ bias,
                                    const int* __restrict__ positions, const float* __restrict__ q_head_w,
                                    const float* __restrict__ k_head_w, float head_w_eps,
                                    const double* __restrict__ inv_freq, double magnitude, const float2* table, int rotary, int pairing,
                                    A* __restrict__ q_out, A* __restrict__ k_out, A* __restrict__ v_out,
                                    A* __restrict__ k_pages, A* __restrict__ v_pages,
                                    const int* __restrict__ dest_rows, int q_heads, int kv_heads, int d, int dv,
                                    int page_size) {
  extern __shared__ float cs[];  // without a table: [rotary / 2] cosines, then as many sines
  const int half = rotary / 2;
  pdl_trigger();
  const int t = blockIdx.x;
  const float2* angles = table != nullptr ? table + static_cast<size_t>(t) * half : nullptr;
  if (table == nullptr) {
    const int pos = positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
      double sn, c;
      sincos(static_cast<double>(pos) * inv_freq[i], &sn, &c);
      cs[i] = static_cast<float>(c * magnitude);
      cs[half + i] = static_cast<float>(sn * magnitude);
    }
    __syncthreads();
  }
  const int dest = k_pages != nullptr ? dest_rows[t] : -1;
  const size_t page = dest >= 0 ? static_cast<size_t>(dest / page_size) : 0;
  const int in_page = dest >= 0 ? dest % page_size : 0;
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const S* row = proj + static_cast<size_t>(t) * stride;
  for (int hd = blockIdx.y * warps + warp; hd < q_heads + 2 * kv_heads; hd += warps * gridDim.y) {
    const bool is_q = hd < q_heads, is_v = hd >= q_heads + kv_heads;
    const int kh = is_q ? 0 : hd - q_heads - (is_v ? kv_heads : 0);
    const int n = is_v ? dv : d;
    const int first = is_v ? (q_heads + kv_heads) * d + kh * dv : hd * d;  // column in the row
    const S* src = row + first;
    const float* add = bias != nullptr ? bias + first : nullptr;
    const float* w = is_v ? nullptr : is_q ? q_head_w : k_head_w;
    float x[kHeadPer];
#pragma unroll
    for (int g = 0; g < kHeadPer / VEC; ++g) {
      const int i = (g * 32 + lane) * VEC;
#pragma unroll
      for (int e = 0; e < VEC; ++e)
        x[g * VEC + e] = i + e < n ? to_f32(src[i + e]) + (add != nullptr ? add[i + e] : 0.f) : 0.f;
    }
    float inv = 1.f;
    if (w != nullptr) {
      float ss = 0.f;
#pragma unroll
      for (int u = 0; u < kHeadPer; ++u) ss = fmaf(x[u], x[u], ss);
      inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(d) + head_w_eps);
    }
    A* packed = is_q ? q_out + (static_cast<size_t>(t) * q_heads + hd) * d
                : is_v ? (v_out != nullptr ? v_out + (static_cast<size_t>(t) * kv_heads + kh) * dv : nullptr)
                       : (k_out != nullptr ? k_out + (static_cast<size_t>(t) * kv_heads + kh) * d : nullptr);
    A* cached = (is_q || dest < 0) ? nullptr
                : (is_v ? v_pages : k_pages) + ((page * kv_heads + kh) * page_size + in_page) * n;
#pragma unroll
    for (int g = 0; g < kHeadPer / VEC; ++g) {
      const int i = (g * 32 + lane) * VEC;
      if (i >= n) continue;
      A y[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const int c = i + e;
        float v = w != nullptr ? (x[g * VEC + e] * inv) * w[c] : x[g * VEC + e];
        if (!is_v && c < rotary) {
          // this element's pair: the partner is read again (it is in L1) and shaped alike
          const int pair = pairing == 0 ? (c < half ? c : c - half) : c >> 1;
          const bool leads = pairing == 0 ? c < half : (c & 1) == 0;
          const int other = pairing == 0 ? (leads ? c + half : c - half) : (leads ? c + 1 : c - 1);
          float p = to_f32(src[other]) + (add != nullptr ? add[other] : 0.f);
          if (w != nullptr) p = (p * inv) * w[other];
          const float2 turn = angles != nullptr ? angles[pair] : make_float2(cs[pair], cs[half + pair]);
          const float co = turn.x, sn = turn.y;
          v = leads ? fmaf(v, co, -__fmul_rn(p, sn)) : fmaf(v, co, __fmul_rn(p, sn));
        }
        y[e] = from_f32<A>(v);
      }
#pragma unroll
      for (int target = 0; target < 2; ++target) {
        A* dst = target == 0 ? packed : cached;
        if (dst == nullptr) continue;
        if constexpr (VEC == 2 && sizeof(A) == 2) {
          *reinterpret_cast<uint32_t*>(dst + i) = *reinterpret_cast<const uint32_t*>(y);
        } else {
#pragma unroll
          for (int e = 0; e < VEC; ++e) dst[i + e] = y[e];
        }
      }
    }
  }
}

template <typename A> __device__ __forceinline__ void store4(A* dst, const float (&y)[4]);
template <> __device__ __forceinline__ void store4<float>(float* dst, const float (&y)[4]) {
  *reinterpret_cast<float4*>(dst) = make_float4(y[0], y[1], y[2], y[3]);
}
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* dst, const float (&y)[4]) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(y[0], y[1]), hi = __floats2bfloat162_rn(y[2], y[3]);
  *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
}

// A thread takes four consecutive columns of the row of token blockIdx.x; `quads` of them make a row.
template <typename A>
__global__ __launch_bounds__(256) void split_rotate_kernel(const float* proj, long long stride, const float* __restrict__ bias,
                                                           const float2* table, int rotary, A* __restrict__ q_out,
                                                           A* __restrict__ k_out, A* __restrict__ v_out,
                                                           A* __restrict__ k_pages, A* __restrict__ v_pages,
                                                           const int* __restrict__ dest_rows, int quads, int q_heads,
                                                           int kv_heads, int d, int dv, int page_size) {
  pdl_trigger();
  const int t = blockIdx.x, col = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
  if (col >= quads * 4) return;
  const int nqk = (q_heads + kv_heads) * d, half = rotary / 2;
  const bool is_v = col >= nqk;
  const int hd = is_v ? (col - nqk) / dv : col / d, c = is_v ? col - nqk - hd * dv : col - hd * d;
  const bool is_q = !is_v && hd < q_heads;
  const int kh = is_v ? hd : hd - q_heads;
  const int dest = !is_q && k_pages != nullptr ? dest_rows[t] : -1;
  const bool turned = !is_v && c < rotary, leads = c < half;
  const int other = leads ? col + half : col - half;  // the partners of a turned quad
  float4 add = make_float4(0.f, 0.f, 0.f, 0.f), add_other = add;
  if (bias != nullptr) {
    add = *reinterpret_cast<const float4*>(bias + col);
    if (turned) add_other = *reinterpret_cast<const float4*>(bias + other);
  }
  pdl_wait();
  const float* row = proj + static_cast<size_t>(t) * stride;
  const float4 x = *reinterpret_cast<const float4*>(row + col);
  float y[4] = {x.x + add.x, x.y + add.y, x.z + add.z, x.w + add.w};
  if (turned) {
    const float4 p = *reinterpret_cast<const float4*>(row + other);
    const float4* turns = reinterpret_cast<const float4*>(table + static_cast<size_t>(t) * half + (leads ? c : c - half));
    const float4 a = turns[0], b = turns[1];  // (cos, sin) of two pairs each
    const float co[4] = {a.x, a.z, b.x, b.z}, sn[4] = {a.y, a.w, b.y, b.w};
    const float q[4] = {p.x + add_other.x, p.y + add_other.y, p.z + add_other.z, p.w + add_other.w};
#pragma unroll
    for (int e = 0; e < 4; ++e)
      y[e] = leads ? fmaf(y[e], co[e], -__fmul_rn(q[e], sn[e])) : fmaf(y[e], co[e], __fmul_rn(q[e], sn[e]));
  }
  if (is_q) {
    store4(q_out + (static_cast<size_t>(t) * q_heads + hd) * d + c, y);
    return;
  }
  const int n = is_v ? dv : d;
  A* packed = is_v ? v_out : k_out;
  if (packed != nullptr) store4(packed + (static_cast<size_t>(t) * kv_heads + kh) * n + c, y);
  if (dest >= 0) {
    const size_t at = (static_cast<size_t>(dest / page_size) * kv_heads + kh) * page_size + dest % page_size;
    store4((is_v ? v_pages : k_pages) + at * n + c, y);
  }
}

}  // namespace

// proj: [tokens, stride], of whose columns the first q_heads * d + kv_heads * (d + dv) are the row;
// float32 or bfloat16 (in_dtype); outputs of out_dtype. bias, taps (float32 [n, row]; + tails, cu_seqlens, seq_of_token, slots), q_norm + k_norm, q_head_w
// + k_head_w (float32 [d] each), inv_freq (double [rotary / 2]) may each be null: that step is then left out. kv_heads 0: queries only.
LRM_API int lrm_shaped_qkv_store(const void* proj, int in_dtype, long long stride, const float* bias, const float* taps, int n,
                                 const float* tails, const int* cu_seqlens, const int* seq_of_token,
                                 const int* slots, const int* positions, const float* q_norm, const float* k_norm,
                                 float row_eps, const float* q_head_w, const float* k_head_w, float head_w_eps,
                                 const double* inv_freq, double magnitude, const float* table, int rotary, int pairing, int head_norm,
                                 float head_eps, void* q_out, void* k_out, void* v_out, void* k_pages, void* v_pages,
                                 const int* dest_rows, int out_dtype, int tokens, int q_heads, int kv_heads, int d,
                                 int dv, int page_size, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (q_heads <= 0 || kv_heads < 0 || d <= 0 || dv < 0 || page_size <= 0 || positions == nullptr) return LRM_BAD_ARGUMENT;
  if (rotary < 0 || rotary > d || rotary % 2 || (rotary > 0 && inv_freq == nullptr && table == nullptr) || (pairing != 0 && pairing != 1))
    return LRM_BAD_ARGUMENT;
  if (inv_freq == nullptr && table == nullptr) rotary = 0;
  const float2* turns = reinterpret_cast<const float2*>(table);
  if ((q_norm != nullptr && kv_heads > 0 && k_norm == nullptr) || (q_norm == nullptr && k_norm != nullptr))
    return LRM_BAD_ARGUMENT;
  if (taps != nullptr && n > 1 && (tails == nullptr || cu_seqlens == nullptr || seq_of_token == nullptr || slots == nullptr))
    return LRM_BAD_ARGUMENT;
  if (k_pages != nullptr && dest_rows == nullptr) return LRM_BAD_ARGUMENT;
  if ((q_head_w == nullptr) != (k_head_w == nullptr)) return LRM_BAD_ARGUMENT;
  const int width = q_heads * d + kv_heads * (d + dv);
  if (stride < width) return LRM_BAD_ARGUMENT;
  const uintptr_t all = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(bias) | reinterpret_cast<uintptr_t>(table) |
                        reinterpret_cast<uintptr_t>(q_out) | reinterpret_cast<uintptr_t>(k_out) | reinterpret_cast<uintptr_t>(v_out) |
                        reinterpret_cast<uintptr_t>(k_pages) | reinterpret_cast<uintptr_t>(v_pages);
  if (taps == nullptr && q_norm == nullptr && q_head_w == nullptr && !head_norm && pairing == 0 && in_dtype == LRM_F32 &&
      (rotary == 0 || table != nullptr) && rotary % 8 == 0 && d % 4 == 0 && dv % 4 == 0 && stride % 4 == 0 && all % 16 == 0) {
    const int quads = width / 4;
    const int threads = quads >= 256 ? 256 : (quads + 31) / 32 * 32;
#define LRM_SPLIT_ROTATE(AT)                                                                                          \
  LRM_LAUNCH((split_rotate_kernel<AT>), dim3(tokens, (quads + threads - 1) / threads), threads, 0, stream,            \
             static_cast<const float*>(proj), stride, bias, turns, rotary, static_cast<AT*>(q_out), static_cast<AT*>(k_out), \
             static_cast<AT*>(v_out), static_cast<AT*>(k_pages), static_cast<AT*>(v_pages), dest_rows, quads, q_heads, \
             kv_heads, d, dv, page_size)
    if (out_dtype == LRM_F32) LRM_SPLIT_ROTATE(float);
    else if (out_dtype == LRM_BF16) LRM_SPLIT_ROTATE(__nv_bfloat16);
    else return LRM_BAD_ARGUMENT;
#undef LRM_SPLIT_ROTATE
    return 0;
  }
  if (taps == nullptr && q_norm == nullptr && !head_norm && d <= 32 * kHeadPer && dv <= 32 * kHeadPer) {
    const int heads = q_heads + 2 * kv_heads;
    const int threads = 32 * (heads < 4 ? heads : heads >= 16 ? 8 : 4);
    // few tokens: a warp per head; many: a CTA per token, which makes its table of angles once
    const dim3 grid(tokens, tokens < 148 ? (heads * 32 + threads - 1) / threads : 1);
    const size_t in_pair = in_dtype == LRM_F32 ? 8 : 4;
    const bool pairs = d % 2 == 0 && dv % 2 == 0 && stride % 2 == 0 && reinterpret_cast<uintptr_t>(proj) % in_pair == 0;
#define LRM_HEADS(ST, AT, V)                                                                                        \
  LRM_LAUNCH((shaped_heads_kernel<ST, AT, V>), grid, threads, sizeof(float) * rotary, stream, static_cast<const ST*>(proj), \
             stride, bias, positions, q_head_w, k_head_w, head_w_eps, inv_freq, magnitude, turns, rotary, pairing, static_cast<AT*>(q_out), \
             static_cast<AT*>(k_out), static_cast<AT*>(v_out), static_cast<AT*>(k_pages), static_cast<AT*>(v_pages), \
             dest_rows, q_heads, kv_heads, d, dv, page_size)
    if (in_dtype == LRM_F32 && out_dtype == LRM_F32) {
      if (pairs) LRM_HEADS(float, float, 2); else LRM_HEADS(float, float, 1);
    } else if (in_dtype == LRM_F32 && out_dtype == LRM_BF16) {
      if (pairs) LRM_HEADS(float, __nv_bfloat16, 2); else LRM_HEADS(float, __nv_bfloat16, 1);
    } else if (in_dtype == LRM_BF16 && out_dtype == LRM_BF16) {
      if (pairs) LRM_HEADS(__nv_bfloat16, __nv_bfloat16, 2); else LRM_HEADS(__nv_bfloat16, __nv_bfloat16, 1);
    } else {
      return LRM_BAD_ARGUMENT;
    }
#undef LRM_HEADS
    return 0;
  }
  const size_t bytes = sizeof(float) * (static_cast<size_t>(width) + rotary);
  if (bytes > 200 * 1024) return LRM_UNSUPPORTED;
#define LRM_SHAPED(ST, AT)                                                                                      \
  do {                                                                                                          \
    static bool raised = false;                                                                                 \
    if (bytes > 48 * 1024 && !raised) {                                                                         \
      cudaError_t e = cudaFuncSetAttribute(shaped_qkv_kernel<ST, AT>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           200 * 1024);                                                         \
      if (e != cudaSuccess) return static_cast<int>(e);                                                         \
      raised = true;                                                                                            \
    }                                                                                                           \
    LRM_LAUNCH((shaped_qkv_kernel<ST, AT>), tokens, width >= 2048 ? 512 : 256, bytes, stream, static_cast<const ST*>(proj), stride, bias, taps, n, \
               tails, cu_seqlens, seq_of_token, slots, positions, q_norm, k_norm, row_eps, q_head_w, k_head_w, head_w_eps, inv_freq, magnitude, turns, rotary, \
               pairing, head_norm, head_eps, static_cast<AT*>(q_out), static_cast<AT*>(k_out),                  \
               static_cast<AT*>(v_out), static_cast<AT*>(k_pages), static_cast<AT*>(v_pages), dest_rows, q_heads, \
               kv_heads, d, dv, page_size);                                                                     \
  } while (0)
  if (in_dtype == LRM_F32 && out_dtype == LRM_F32)
    LRM_SHAPED(float, float);
  else if (in_dtype == LRM_F32 && out_dtype == LRM_BF16)
    LRM_SHAPED(float, __nv_bfloat16);
  else if (in_dtype == LRM_BF16 && out_dtype == LRM_BF16)
    LRM_SHAPED(__nv_bfloat16, __nv_bfloat16);
  else
    return LRM_BAD_ARGUMENT;
#undef LRM_SHAPED
  return 0;
}
