// What a time-mixing layer needs around its products and its scan (recurrent_scan.cu):
//
//  * token_mixes: several mixes of a token's row with the row before it, out[s, t] = h[t] + (h[t - 1] -
//    h[t]) * mix[s], in one pass over the rows, as the inputs of several projections;
//  * decay_product: the decay per head and key channel from a low-rank product, g = exp(-exp(W tanh(z) +
//    bias)): the tanh on the way into the product, the exponentials on its sums. bfloat16 runs the
//    product on mma.sync with the tanh rounded to bfloat16, float32 in true float32.
#include "common.cuh"

namespace {

// One CTA per (token, range of channels); the thread that reads the kept row of a sequence for its first
// token of the step writes the sequence's newest row there (see token_shift.cu).
template <typename A, int VEC>
__global__ void token_mixes_kernel(const A* h, const float* __restrict__ mix, int mixes, float* last,
                                   A* __restrict__ out, const int* __restrict__ cu_seqlens,
                                   const int* __restrict__ seq_of_token, const int* __restrict__ slots, int width,
                                   size_t plane) {
  pdl_trigger();
  const int t = blockIdx.x;
  const int b = seq_of_token[t], local = t - cu_seqlens[b], slot = slots[b];
  const int newest = cu_seqlens[b + 1] - 1;
  pdl_wait();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (c >= width) return;
  const A* row = h + static_cast<size_t>(t) * width + c;
  float* kept = (local == 0 && slot >= 0) ? last + static_cast<size_t>(slot) * width + c : nullptr;
  float x[VEC], step[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) {
    x[e] = to_f32(row[e]);
    const float before = local > 0 ? to_f32(row[e - width]) : kept != nullptr ? kept[e] : 0.f;
    step[e] = before - x[e];
    if (kept != nullptr) kept[e] = to_f32(h[static_cast<size_t>(newest) * width + c + e]);
  }
  for (int s = 0; s < mixes; ++s) {
    const float* m = mix + static_cast<size_t>(s) * width + c;
    A y[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = from_f32<A>(fmaf(step[e], m[e], x[e]));
    A* dst = out + s * plane + static_cast<size_t>(t) * width + c;
    if constexpr (VEC == 4 && sizeof(A) == 2) {
      *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(y);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) dst[e] = y[e];
    }
  }
}

__device__ __forceinline__ float decay_of(float z) { return expf(-expf(z)); }

constexpr int kM = 64, kN = 64;  // tokens x channels of a CTA's tile

// true float32: 256 threads, 4 x 4 results each, k ascending
__global__ __launch_bounds__(256) void decay_product_f32_kernel(const float* z, long long stride,
                                                                const float* __restrict__ W,
                                                                const float* __restrict__ bias,
                                                                float* __restrict__ g, int M, int N, int K) {
  constexpr int BK = 16;
  __shared__ float Zs[BK][kM + 4], Ws[BK][kN + 4];
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4, m0 = blockIdx.y * kM, n0 = blockIdx.x * kN;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = tid + i * 256, r = idx >> 4, c = idx & 15;
      Zs[c][r] = (m0 + r < M && k0 + c < K) ? tanhf(z[static_cast<size_t>(m0 + r) * stride + k0 + c]) : 0.f;
      Ws[c][r] = (n0 + r < N && k0 + c < K) ? W[static_cast<size_t>(n0 + r) * K + k0 + c] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < BK; ++kk)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(Zs[kk][ty * 4 + i], Ws[kk][tx * 4 + j], acc[i][j]);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) g[static_cast<size_t>(m) * N + n] = decay_of(acc[i][j] + bias[n]);
    }
}

__device__ __forceinline__ void mma_bf16_16816(float (&c)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 "
      "{%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}

// four warps, 32 tokens x 32 channels each
__global__ __launch_bounds__(128) void decay_product_bf16_kernel(const float* z, long long stride,
                                                                 const __nv_bfloat16* __restrict__ W,
                                                                 const float* __restrict__ bias,
                                                                 float* __restrict__ g, int M, int N, int K,
                                                                 int fours) {
  constexpr int BK = 64, PITCH = BK + 8;
  __shared__ __align__(16) __nv_bfloat16 Zs[kM][PITCH], Ws[kN][PITCH];
  pdl_trigger();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, t = lane & 3;
  const int wm = (warp >> 1) * 32, wn = (warp & 1) * 32, m0 = blockIdx.y * kM, n0 = blockIdx.x * kN;
  float acc[2][4][4] = {};
  for (int k0 = 0; k0 < K; k0 += BK) {
    if (fours) {
      for (int idx = tid; idx < kN * BK / 4; idx += 128) {  // a weight: needs no wait
        const int r = idx / (BK / 4), c = idx % (BK / 4) * 4;
        uint2 w = make_uint2(0u, 0u);
        if (n0 + r < N && k0 + c < K) w = *reinterpret_cast<const uint2*>(W + static_cast<size_t>(n0 + r) * K + k0 + c);
        *reinterpret_cast<uint2*>(&Ws[r][c]) = w;
      }
      if (k0 == 0) pdl_wait();
      for (int idx = tid; idx < kM * BK / 4; idx += 128) {
        const int r = idx / (BK / 4), c = idx % (BK / 4) * 4;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (m0 + r < M && k0 + c < K) v = *reinterpret_cast<const float4*>(z + static_cast<size_t>(m0 + r) * stride + k0 + c);
        __nv_bfloat162 lo = __floats2bfloat162_rn(tanhf(v.x), tanhf(v.y)), hi = __floats2bfloat162_rn(tanhf(v.z), tanhf(v.w));
        *reinterpret_cast<uint2*>(&Zs[r][c]) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
      }
    } else {
      for (int idx = tid; idx < kN * BK; idx += 128) {
        const int r = idx / BK, c = idx % BK;
        Ws[r][c] = (n0 + r < N && k0 + c < K) ? W[static_cast<size_t>(n0 + r) * K + k0 + c] : __float2bfloat16_rn(0.f);
      }
      if (k0 == 0) pdl_wait();
      for (int idx = tid; idx < kM * BK; idx += 128) {
        const int r = idx / BK, c = idx % BK;
        Zs[r][c] = __float2bfloat16_rn((m0 + r < M && k0 + c < K) ? tanhf(z[static_cast<size_t>(m0 + r) * stride + k0 + c]) : 0.f);
      }
    }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < BK; ks += 16) {
      uint32_t a[2][4], b[4][2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = wm + i * 16 + gq;
        a[i][0] = *reinterpret_cast<const uint32_t*>(&Zs[r][ks + 2 * t]);
        a[i][1] = *reinterpret_cast<const uint32_t*>(&Zs[r + 8][ks + 2 * t]);
        a[i][2] = *reinterpret_cast<const uint32_t*>(&Zs[r][ks + 2 * t + 8]);
        a[i][3] = *reinterpret_cast<const uint32_t*>(&Zs[r + 8][ks + 2 * t + 8]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = wn + j * 8 + gq;
        b[j][0] = *reinterpret_cast<const uint32_t*>(&Ws[n][ks + 2 * t]);
        b[j][1] = *reinterpret_cast<const uint32_t*>(&Ws[n][ks + 2 * t + 8]);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) mma_bf16_16816(acc[i][j], a[i], b[j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int m = m0 + wm + i * 16 + gq + 8 * half, n = n0 + wn + j * 8 + 2 * t;
        if (m >= M || n >= N) continue;
        float* dst = g + static_cast<size_t>(m) * N + n;
        const float first = decay_of(acc[i][j][2 * half] + bias[n]);
        if (N % 2 == 0) {
          *reinterpret_cast<float2*>(dst) = make_float2(first, decay_of(acc[i][j][2 * half + 1] + bias[n + 1]));
        } else {
          dst[0] = first;
          if (n + 1 < N) dst[1] = decay_of(acc[i][j][2 * half + 1] + bias[n + 1]);
        }
      }
}

}  // namespace

// h [tokens, width], out [mixes, plane / width rows or more, width] of `dtype` (planes `plane` elements
// apart); mix float32 [mixes, width]; last float32 [slots, width].
LRM_API int lrm_token_mixes(const void* h, int dtype, const float* mix, int mixes, float* last, void* out,
                            long long plane, const int* cu_seqlens, const int* seq_of_token, const int* slots,
                            int tokens, int width, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (width <= 0 || mixes <= 0 || mix == nullptr || last == nullptr || plane < static_cast<long long>(tokens) * width)
    return LRM_BAD_ARGUMENT;
  const bool four = width % 4 == 0 && plane % 4 == 0 && reinterpret_cast<uintptr_t>(out) % 8 == 0;
  const int groups = four ? width / 4 : width;
  const int threads = groups >= 256 ? 256 : ((groups + 31) / 32) * 32;
  const dim3 grid(tokens, (groups + threads - 1) / threads);
  if (grid.y > 65535) return LRM_UNSUPPORTED;
#define LRM_MIXES(AT, V)                                                                                             \
  LRM_LAUNCH((token_mixes_kernel<AT, V>), grid, threads, 0, stream, static_cast<const AT*>(h), mix, mixes, last,      \
             static_cast<AT*>(out), cu_seqlens, seq_of_token, slots, width, static_cast<size_t>(plane))
  if (dtype == LRM_F32) {
    if (four) LRM_MIXES(float, 4); else LRM_MIXES(float, 1);
  } else if (dtype == LRM_BF16) {
    if (four) LRM_MIXES(__nv_bfloat16, 4); else LRM_MIXES(__nv_bfloat16, 1);
  } else {
    return LRM_BAD_ARGUMENT;
  }
#undef LRM_MIXES
  return 0;
}

// z: float32 columns of a [M, stride] activation (pointer at the first); W [N, K] of w_dtype (float32:
// true float32; bfloat16: tensor cores); bias float32 [N]; g float32 [M, N].
LRM_API int lrm_decay_product(const float* z, long long stride, const void* W, int w_dtype, const float* bias, float* g,
                              int M, int N, int K, cudaStream_t stream) {
  if (M <= 0 || N <= 0) return 0;
  if (K <= 0 || stride < K || z == nullptr || W == nullptr || bias == nullptr) return LRM_BAD_ARGUMENT;
  const dim3 grid((N + kN - 1) / kN, (M + kM - 1) / kM);
  if (grid.y > 65535) return LRM_UNSUPPORTED;
  if (w_dtype == LRM_F32)
    LRM_LAUNCH(decay_product_f32_kernel, grid, 256, 0, stream, z, stride, static_cast<const float*>(W), bias, g, M, N, K);
  else if (w_dtype == LRM_BF16)
    LRM_LAUNCH(decay_product_bf16_kernel, grid, 128, 0, stream, z, stride, static_cast<const __nv_bfloat16*>(W), bias, g,
               M, N, K,
               K % 4 == 0 && stride % 4 == 0 && reinterpret_cast<uintptr_t>(z) % 16 == 0 &&
                   reinterpret_cast<uintptr_t>(W) % 8 == 0);
  else
    return LRM_BAD_ARGUMENT;
  return 0;
}
