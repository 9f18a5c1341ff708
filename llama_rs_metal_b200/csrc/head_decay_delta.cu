// Inputs of the delta rule with one decay per head and token (the scan itself is the state scan of
// recurrent_scan.cu). From the fused projection row [.. q (G d) | k (G d) | v (H dv) .. b (H) .. a (H) ..]:
//   q, k, v pass a short causal convolution over time per channel (taps [n, C], the last row the current
//   token's, no bias, zeros before the sequence's start) and SiLU; every q and k head becomes a unit
//   vector, x / sqrt(sum x^2 + unit_eps), q also times q_scale;
//   step  = sigmoid(b)                                      per head
//   decay = exp(-rate_h softplus(a + dt_bias_h))            per head, rate = exp(A_log) made by the caller
// all in float32. A warp takes one head (of q, k or v) of one token; one more takes the token's scalars.
// Inputs before the step's first token come from the sequence's tail [n - 1, C]. In a step of one token
// per sequence the warp that read a channel's tail also moves it on; longer steps leave that to
// conv_tail_update. The projection is the output of the kernel before: it is read through a plain pointer.
#include "common.cuh"

namespace {

template <typename S, int PER>
__global__ void head_decay_delta_prepare_kernel(const S* proj, long long stride, int conv_off, int b_off, int a_off,
                                                const float* __restrict__ dt_bias, const float* __restrict__ rate,
                                                const float* __restrict__ taps, int n, float* tails,
                                                const int* __restrict__ cu_seqlens,
                                                const int* __restrict__ seq_of_token, const int* __restrict__ slots,
                                                float* __restrict__ qf, float* __restrict__ kf,
                                                float* __restrict__ vf, float* __restrict__ decay,
                                                float* __restrict__ step, int H, int G, int d, int dv, float unit_eps,
                                                float q_scale, int one_each) {
  pdl_trigger();
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  const int seg = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int C = 2 * G * d + H * dv;
  const int b = seq_of_token[t], local = t - cu_seqlens[b], slot = slots[b];
  pdl_wait();
  if (seg > 2 * G + H) return;
  const S* row = proj + static_cast<size_t>(t) * stride;
  if (seg == 2 * G + H) {
    for (int h = lane; h < H; h += 32) {
      const size_t at = static_cast<size_t>(t) * H + h;
      step[at] = 1.0f / (1.0f + expf(-to_f32(row[b_off + h])));
      const float z = to_f32(row[a_off + h]) + dt_bias[h];
      decay[at] = expf(-rate[h] * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)))));
    }
    return;
  }
  const bool unit = seg < 2 * G;
  const int size = unit ? d : dv, first = unit ? seg * d : 2 * G * d + (seg - 2 * G) * dv;
  float* dst = seg < G ? qf + (static_cast<size_t>(t) * G + seg) * d
               : unit ? kf + (static_cast<size_t>(t) * G + seg - G) * d
                      : vf + (static_cast<size_t>(t) * H + seg - 2 * G) * dv;
  float* tail = (slot >= 0 && n > 1) ? tails + static_cast<size_t>(slot) * (n - 1) * C : nullptr;
  float y[PER], now[PER];
#pragma unroll
  for (int u = 0; u < PER; ++u) y[u] = 0.f;
  for (int back = n - 1; back >= 0; --back) {  // oldest input first; a tap's loads are all under way together
    const int at = local - back;
    const S* input = at >= 0 ? row + conv_off + first - static_cast<long long>(back) * stride : nullptr;
    const float* kept = (at < 0 && tail != nullptr) ? tail + static_cast<size_t>(n - 1 + at) * C + first : nullptr;
    const float* tap = taps + static_cast<size_t>(n - 1 - back) * C + first;
#pragma unroll
    for (int u = 0; u < PER; ++u) {
      const int i = lane + 32 * u;
      if (i < size) {
        now[u] = input != nullptr ? to_f32(input[i]) : kept != nullptr ? kept[i] : 0.f;
        y[u] = fmaf(tap[i], now[u], y[u]);
      }
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < PER; ++u) {
    const int i = lane + 32 * u, c = first + i;
    if (i < size && one_each && tail != nullptr) {
      for (int s = 0; s + 1 < n - 1; ++s)
        tail[static_cast<size_t>(s) * C + c] = tail[static_cast<size_t>(s + 1) * C + c];
      tail[static_cast<size_t>(n - 2) * C + c] = now[u];  // the last input read is the token's own
    }
    y[u] = y[u] / (1.0f + expf(-y[u]));
    ss = fmaf(y[u], y[u], ss);
  }
  float factor = 1.f;
  if (unit) factor = (seg < G ? q_scale : 1.0f) / sqrtf(warp_sum(ss) + unit_eps);
#pragma unroll
  for (int u = 0; u < PER; ++u) {
    const int i = lane + 32 * u;
    if (i < size) dst[i] = y[u] * factor;
  }
}

}  // namespace

// proj [tokens, stride] float32 or bfloat16. one_each: every sequence of the step brings exactly one
// token (the tails are then rewritten here). -> qf, kf [T, G, d], vf [T, H, dv], decay, step [T, H].
LRM_API int lrm_head_decay_delta_prepare(const void* proj, int dtype, long long stride, int conv_off, int b_off,
                                         int a_off, const float* dt_bias, const float* rate, const float* taps, int n,
                                         float* tails, const int* cu_seqlens, const int* seq_of_token,
                                         const int* slots, float* qf, float* kf, float* vf, float* decay, float* step,
                                         int tokens, int H, int G, int d, int dv, float unit_eps, float q_scale,
                                         int one_each, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || d <= 0 || dv <= 0 || n <= 0 || (n > 1 && tails == nullptr)) return LRM_BAD_ARGUMENT;
  const int widest = d > dv ? d : dv, segments = 2 * G + H + 1, warps = 4;
  if (widest > 1024 || (segments + warps - 1) / warps > 65535) return LRM_UNSUPPORTED;
  const dim3 grid(tokens, (segments + warps - 1) / warps);
#define LRM_PREPARE(ST, PER)                                                                                     \
  LRM_LAUNCH((head_decay_delta_prepare_kernel<ST, PER>), grid, warps * 32, 0, stream, static_cast<const ST*>(proj), \
             stride, conv_off, b_off, a_off, dt_bias, rate, taps, n, tails, cu_seqlens, seq_of_token, slots, qf, kf, \
             vf, decay, step, H, G, d, dv, unit_eps, q_scale, one_each)
#define LRM_PREPARE_BY_SIZE(ST)             \
  do {                                      \
    if (widest <= 64) LRM_PREPARE(ST, 2);   \
    else if (widest <= 128) LRM_PREPARE(ST, 4); \
    else if (widest <= 256) LRM_PREPARE(ST, 8); \
    else LRM_PREPARE(ST, 32);               \
  } while (0)
  if (dtype == LRM_F32)
    LRM_PREPARE_BY_SIZE(float);
  else if (dtype == LRM_BF16)
    LRM_PREPARE_BY_SIZE(__nv_bfloat16);
  else
    return LRM_BAD_ARGUMENT;
#undef LRM_PREPARE_BY_SIZE
#undef LRM_PREPARE
  return 0;
}
