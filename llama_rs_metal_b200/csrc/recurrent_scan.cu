// The state scans with a plain decay (see recurrent_scan.cuh), the read-out's norm and gate, and the
// inputs of retention and of the gated delta rule.
#include "recurrent_scan.cuh"

int g_scan_rows = 16;

extern "C" int lrm_scan_gated_delta(const float* q, const float* k, const float* v, const float* g, const float* beta,
                                    float* state, float* out, const int* cu_seqlens, const int* slots, int seqs, int H,
                                    int KH, int d, int dv, int tokens, cudaStream_t stream);  // recurrent_scan_delta.cu

namespace {

// --------------------------------------------------------------------------- read-out: norm and gate per head
// out[t, h, :] = o / sqrt(mean(o^2) + eps) * w * act(gate[t, h, :]) * out_scale; w and gate optional.
// A head's row of `o` has o_stride floats of which the first dv are read (o_stride > dv: the scan
// carried more columns). w is shared by the heads (w_stride 0) or one row per head (w_stride dv).
// With `floor` [T, H] the head is first divided by max(|o[dv]|, floor[t, h]) + den_eps: o's column dv
// then holds the read-out of a normalizer that went through the scan as one more value column.
template <typename A, typename G>
__global__ void head_norm_gate_kernel(const float* __restrict__ o, int o_stride, const float* __restrict__ weight,
                                      int w_stride, const float* __restrict__ floor, float den_eps,
                                      const G* __restrict__ gate, long long gate_stride, int gate_act,
                                      A* __restrict__ out, long long out_stride, int H, int dv, float eps,
                                      float out_scale) {
  __shared__ float scratch[32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y;
  const float* row = o + (static_cast<size_t>(t) * H + h) * o_stride;
  float under = 1.0f;
  if (floor != nullptr) under = 1.0f / (fmaxf(fabsf(row[dv]), floor[static_cast<size_t>(t) * H + h]) + den_eps);
  float ss = 0.f;
  for (int j = threadIdx.x; j < dv; j += blockDim.x) {
    const float v = row[j] * under;
    ss = fmaf(v, v, ss);
  }
  const float total = block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(total / static_cast<float>(dv) + eps);
  for (int j = threadIdx.x; j < dv; j += blockDim.x) {
    float y = (row[j] * under) * inv;
    if (weight != nullptr) y *= weight[h * w_stride + j];
    if (gate != nullptr) {
      const float z = to_f32(gate[static_cast<size_t>(t) * gate_stride + h * dv + j]);
      const float sig = 1.0f / (1.0f + expf(-z));
      y *= gate_act == 1 ? z * sig : sig;
    }
    out[static_cast<size_t>(t) * out_stride + h * dv + j] = from_f32<A>(y * out_scale);
  }
}

// The same with a warp per (token, head), for heads of up to 32 * PER values, which stay in registers.
template <typename A, typename G, int PER>
__global__ void head_norm_gate_warp_kernel(const float* o, int o_stride, const float* __restrict__ weight,
                                           int w_stride, const float* floor, float den_eps, const G* gate,
                                           long long gate_stride, int gate_act, A* __restrict__ out,
                                           long long out_stride, long long heads, int H, int dv, float eps,
                                           float out_scale) {
  pdl_trigger();
  pdl_wait();
  const long long idx = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (idx >= heads) return;
  const int lane = threadIdx.x & 31, h = static_cast<int>(idx % H);
  const size_t t = static_cast<size_t>(idx / H);
  const float* row = o + idx * o_stride;
  float under = 1.0f;
  if (floor != nullptr) under = 1.0f / (fmaxf(fabsf(row[dv]), floor[idx]) + den_eps);
  float v[PER], z[PER];
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < PER; ++u) {
    const int j = lane + 32 * u;
    v[u] = j < dv ? row[j] * under : 0.f;
    z[u] = (gate != nullptr && j < dv) ? to_f32(gate[t * gate_stride + h * dv + j]) : 0.f;
    ss = fmaf(v[u], v[u], ss);
  }
  const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(dv) + eps);
#pragma unroll
  for (int u = 0; u < PER; ++u) {
    const int j = lane + 32 * u;
    if (j >= dv) continue;
    float y = v[u] * inv;
    if (weight != nullptr) y *= weight[h * w_stride + j];
    if (gate != nullptr) {
      const float sig = 1.0f / (1.0f + expf(-z[u]));
      y *= gate_act == 1 ? z[u] * sig : sig;
    }
    out[t * out_stride + h * dv + j] = from_f32<A>(y * out_scale);
  }
}

// --------------------------------------------------------------------------- retention: rotation and key scale
// From the fused projection row [.. q (H d) .. k (H d) .. v (H dv) ..]: q and k of every head are
// rotated on their first `rotary` dimensions (i paired with i + rotary/2, angle = float(position) *
// inv_freq[i], one float32 product), k is multiplied by k_scale after the rotation, v is widened.
template <typename A>
__global__ void retention_prepare_kernel(const A* __restrict__ proj, long long stride, int q_off, int k_off,
                                         int v_off, const int* __restrict__ positions,
                                         const float* __restrict__ inv_freq, int rotary, float k_scale,
                                         float* __restrict__ qf, float* __restrict__ kf,
                                         float* __restrict__ vf, int H, int d, int dv) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y;
  const A* row = proj + static_cast<size_t>(t) * stride;
  const float fpos = static_cast<float>(positions[t]);
  const int half = rotary / 2;
  const size_t o = (static_cast<size_t>(t) * H + h) * d;
  for (int i = threadIdx.x; i < d; i += blockDim.x) {
    const A* qh = row + q_off + h * d;
    const A* kh = row + k_off + h * d;
    float yq = to_f32(qh[i]), yk = to_f32(kh[i]);
    if (i < rotary) {
      const int pair = i < half ? i : i - half;
      const float angle = __fmul_rn(fpos, inv_freq[pair]);
      float sn, cs;
      sincosf(angle, &sn, &cs);
      if (i < half) {  // first of the pair: x cos - partner sin
        yq = fmaf(yq, cs, -__fmul_rn(to_f32(qh[i + half]), sn));
        yk = fmaf(yk, cs, -__fmul_rn(to_f32(kh[i + half]), sn));
      } else {         // second of the pair: x cos + partner sin
        yq = fmaf(yq, cs, __fmul_rn(to_f32(qh[i - half]), sn));
        yk = fmaf(yk, cs, __fmul_rn(to_f32(kh[i - half]), sn));
      }
    }
    qf[o + i] = yq;
    kf[o + i] = yk * k_scale;
  }
  for (int jn = threadIdx.x; jn < dv; jn += blockDim.x)
    vf[(static_cast<size_t>(t) * H + h) * dv + jn] = to_f32(row[v_off + h * dv + jn]);
}

// --------------------------------------------------------------------------- gated delta rule: inputs
// One CTA per (token, segment). Segments: G query heads, G key heads, H value heads (short causal
// convolution over time per channel, then SiLU; q and k then made unit vectors per head, q also
// times q_scale), H heads of decays g = exp(-rate_h softplus(a + dt_bias)), and one of step sizes
// b = sigmoid(.). The convolution's channels are the columns conv_off .. conv_off + C of the
// projection row in the order q | k | v; taps [C, n] with the last column the current token's;
// inputs before the step's first token come from the sequence's tail [n - 1, C] in the state
// storage (zeros at the start of a sequence).
template <typename A>
__device__ __forceinline__ float conv_silu(const A* __restrict__ proj, long long stride, int column, int c,
                                           int t, int local, const float* __restrict__ taps, int n,
                                           const float* __restrict__ tail, int C) {
  float acc = 0.f;
  for (int back = n - 1; back >= 0; --back) {  // oldest input first
    const int at = local - back;
    float x;
    if (at >= 0)
      x = to_f32(proj[static_cast<size_t>(t - back) * stride + column]);
    else
      x = tail != nullptr ? tail[static_cast<size_t>(n - 1 + at) * C + c] : 0.f;
    acc = fmaf(taps[static_cast<size_t>(c) * n + (n - 1 - back)], x, acc);
  }
  return acc / (1.0f + expf(-acc));
}

template <typename A>
__global__ void delta_prepare_kernel(const A* __restrict__ proj, long long stride, int conv_off, int b_off,
                                     const float* __restrict__ a, long long a_stride,
                                     const float* __restrict__ dt_bias, const float* __restrict__ rate, const float* __restrict__ taps, int n,
                                     const float* __restrict__ tails, const int* __restrict__ cu_seqlens,
                                     const int* __restrict__ seq_of_token, const int* __restrict__ slots,
                                     float* __restrict__ qf, float* __restrict__ kf, float* __restrict__ vf,
                                     float* __restrict__ gf, float* __restrict__ bf, int H, int G, int d,
                                     int dv, float unit_eps, float q_scale) {
  __shared__ float scratch[32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, seg = blockIdx.y;
  const int C = 2 * G * d + H * dv;
  if (seg < 2 * G + H) {
    const int b = seq_of_token[t], local = t - cu_seqlens[b], slot = slots[b];
    const float* tail = slot >= 0 ? tails + static_cast<size_t>(slot) * (n - 1) * C : nullptr;
    if (seg < 2 * G) {  // a query or key head: convolution, SiLU, unit vector
      const int first = seg * d;  // q heads then k heads are contiguous channels
      float* dst = (seg < G ? qf + (static_cast<size_t>(t) * G + seg) * d
                            : kf + (static_cast<size_t>(t) * G + seg - G) * d);
      float ss = 0.f;
      // a thread keeps its channels' values between the two passes (d <= 8 * blockDim.x)
      float mine[8];
      int cnt = 0;
      for (int i = threadIdx.x; i < d; i += blockDim.x, ++cnt) {
        const float y = conv_silu(proj, stride, conv_off + first + i, first + i, t, local, taps, n, tail, C);
        mine[cnt] = y;
        ss = fmaf(y, y, ss);
      }
      const float total = block_sum(ss, scratch);
      const float inv = (seg < G ? q_scale : 1.0f) / sqrtf(total + unit_eps);
      cnt = 0;
      for (int i = threadIdx.x; i < d; i += blockDim.x, ++cnt) dst[i] = mine[cnt] * inv;
    } else {
      const int hv = seg - 2 * G, first = 2 * G * d + hv * dv;
      for (int i = threadIdx.x; i < dv; i += blockDim.x)
        vf[(static_cast<size_t>(t) * H + hv) * dv + i] =
            conv_silu(proj, stride, conv_off + first + i, first + i, t, local, taps, n, tail, C);
    }
  } else if (seg < 2 * G + 2 * H) {
    const int hd = seg - 2 * G - H;
    const float r = rate[hd];
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
      const size_t at = (static_cast<size_t>(t) * H + hd) * d + i;
      const float z = a[static_cast<size_t>(t) * a_stride + hd * d + i] + dt_bias[hd * d + i];
      const float sp = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
      gf[at] = expf(-r * sp);
    }
  } else {
    for (int hb = threadIdx.x; hb < H; hb += blockDim.x) {
      const float z = to_f32(proj[static_cast<size_t>(t) * stride + b_off + hb]);
      bf[static_cast<size_t>(t) * H + hb] = 1.0f / (1.0f + expf(-z));
    }
  }
}

// After a step: every sequence's tail becomes the last n - 1 convolution inputs it has seen.
// One thread per (sequence, channel), entries ascending: entry s takes input number
// m - (n - 1) + s of the step's m tokens, or, when that is before the step, the old entry s + m,
// which lies above every entry written so far.
template <typename A>
__global__ void conv_tail_update_kernel(const A* __restrict__ proj, long long stride, int conv_off, int C,
                                        int n, float* __restrict__ tails,
                                        const int* __restrict__ cu_seqlens, const int* __restrict__ slots) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int slot = slots[b];
  if (c >= C || slot < 0) return;
  const int start = cu_seqlens[b], m = cu_seqlens[b + 1] - start;
  float* tail = tails + static_cast<size_t>(slot) * (n - 1) * C;
  for (int s = 0; s < n - 1; ++s) {
    const int at = m - (n - 1) + s;
    tail[static_cast<size_t>(s) * C + c] =
        at >= 0 ? to_f32(proj[static_cast<size_t>(start + at) * stride + conv_off + c])
                : tail[static_cast<size_t>(s + m) * C + c];
  }
}

}  // namespace

// Tuning: the most rows of a state column one thread holds (4, 8, 16, 32 or 64; more rows mean fewer
// parts to add up by shuffles and longer chains of sums per thread). Returns the value in force.
LRM_API int lrm_linear_state_scan_rows(int rows) {
  if (rows == 4 || rows == 8 || rows == 16 || rows == 32 || rows == 64) g_scan_rows = rows;
  return g_scan_rows;
}

// q, k float32 [T, KH, d]; v float32 [T, H, dv]; out float32 [T, H, dv]; state float32
// [slots, H, d, dv]. Without `g`: plain decay per head (head_decay [H]) or, when that is null, per
// head and token (`beta` [T, H] holds the decays); with it: the gated delta rule (g [T, H, d], beta
// [T, H]).
LRM_API int lrm_linear_state_scan(const float* q, const float* k, const float* v, const float* g,
                                  const float* head_decay, const float* beta, float* state, float* out,
                                  const int* cu_seqlens, const int* slots, int seqs, int H, int KH, int d,
                                  int dv, int tokens, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (H <= 0 || KH <= 0 || H % KH || d <= 0 || dv <= 0 || seqs > 65535 || H > 65535) return LRM_BAD_ARGUMENT;
  if (d > 2048) return LRM_UNSUPPORTED;
  if (g != nullptr) {
    if (beta == nullptr) return LRM_BAD_ARGUMENT;
    return lrm_scan_gated_delta(q, k, v, g, beta, state, out, cu_seqlens, slots, seqs, H, KH, d, dv, tokens, stream);
  }
  if (head_decay == nullptr) {  // one decay per head and token, where beta would be
    if (beta == nullptr) return LRM_BAD_ARGUMENT;
    return dispatch_scan<2>(q, k, v, nullptr, nullptr, beta, nullptr, nullptr, state, out, cu_seqlens, slots, seqs, H, KH, d, dv, stream, Rows{tokens});
  }
  return dispatch_scan<0>(q, k, v, nullptr, head_decay, nullptr, nullptr, nullptr, state, out, cu_seqlens, slots, seqs, H, KH, d,
                          dv, stream, Rows{tokens});
}

// `gate` (type gate_dtype, may be null) is read at gate[t * gate_stride + h * dv + j]; o at
// o[(t * H + h) * o_stride + j]; weight at weight[h * w_stride + j]; floor (may be null) at [t * H + h];
// the result goes to out[t * out_stride + h * dv + j].
LRM_API int lrm_head_norm_gate(const float* o, int o_stride, const float* weight, int w_stride, const float* floor,
                               float den_eps, const void* gate, int gate_dtype, long long gate_stride, int gate_act,
                               void* out, int dtype, int tokens, int H, int dv, float eps, float out_scale,
                               long long out_stride, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (out_stride < static_cast<long long>(H) * dv) return LRM_BAD_ARGUMENT;
  if (H <= 0 || H > 65535 || dv <= 0 || (gate != nullptr && gate_act != 1 && gate_act != 2)) return LRM_BAD_ARGUMENT;
  if (o_stride < dv || (floor != nullptr && o_stride <= dv) || (w_stride != 0 && w_stride != dv)) return LRM_BAD_ARGUMENT;
  const int threads = dv >= 256 ? 256 : ((dv + 31) / 32) * 32;
  const dim3 grid(tokens, H);
  const long long heads = static_cast<long long>(tokens) * H;
#define LRM_HEAD_WARP(AT, GT, PER)                                                                          \
  LRM_LAUNCH((head_norm_gate_warp_kernel<AT, GT, PER>), static_cast<unsigned>((heads + 3) / 4), 128, 0, stream, o, \
             o_stride, weight, w_stride, floor, den_eps, static_cast<const GT*>(gate), gate_stride, gate_act, \
             static_cast<AT*>(out), out_stride, heads, H, dv, eps, out_scale)
#define LRM_HEAD_NORM(AT, GT)                                                                              \
  if (dv <= 64) LRM_HEAD_WARP(AT, GT, 2);                                                                  \
  else if (dv <= 128) LRM_HEAD_WARP(AT, GT, 4);                                                            \
  else if (dv <= 256) LRM_HEAD_WARP(AT, GT, 8);                                                            \
  else                                                                                                     \
  LRM_LAUNCH((head_norm_gate_kernel<AT, GT>), grid, threads, 0, stream, o, o_stride, weight, w_stride, floor,    \
             den_eps, static_cast<const GT*>(gate), gate_stride, gate_act, static_cast<AT*>(out), out_stride, H, dv, eps, \
             out_scale)
  if (dtype == LRM_F32 && gate_dtype == LRM_F32) {
    LRM_HEAD_NORM(float, float);
  } else if (dtype == LRM_F32 && gate_dtype == LRM_BF16) {
    LRM_HEAD_NORM(float, __nv_bfloat16);
  } else if (dtype == LRM_BF16 && gate_dtype == LRM_F32) {
    LRM_HEAD_NORM(__nv_bfloat16, float);
  } else if (dtype == LRM_BF16 && gate_dtype == LRM_BF16) {
    LRM_HEAD_NORM(__nv_bfloat16, __nv_bfloat16);
  } else {
    return LRM_BAD_ARGUMENT;
  }
#undef LRM_HEAD_WARP
#undef LRM_HEAD_NORM
  return 0;
}

LRM_API int lrm_retention_prepare(const void* proj, int dtype, long long stride, int q_off, int k_off, int v_off,
                                  const int* positions, const float* inv_freq, int rotary, float k_scale,
                                  float* qf, float* kf, float* vf, int tokens, int H, int d, int dv,
                                  cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (H <= 0 || H > 65535 || d <= 0 || dv <= 0 || rotary < 0 || rotary > d || rotary % 2 ||
      (rotary > 0 && inv_freq == nullptr))
    return LRM_BAD_ARGUMENT;
  const dim3 grid(tokens, H);
  const int widest = d > dv ? d : dv;
  const int threads = widest >= 256 ? 256 : ((widest + 31) / 32) * 32;
  if (dtype == LRM_F32)
    LRM_LAUNCH(retention_prepare_kernel<float>, grid, threads, 0, stream, static_cast<const float*>(proj), stride,
               q_off, k_off, v_off, positions, inv_freq, rotary, k_scale, qf, kf, vf, H, d, dv);
  else if (dtype == LRM_BF16)
    LRM_LAUNCH(retention_prepare_kernel<__nv_bfloat16>, grid, threads, 0, stream,
               static_cast<const __nv_bfloat16*>(proj), stride, q_off, k_off, v_off, positions, inv_freq, rotary,
               k_scale, qf, kf, vf, H, d, dv);
  else
    return LRM_BAD_ARGUMENT;
  return 0;
}

// Every sequence's tail [slots, n - 1, C] becomes the last n - 1 inputs (columns conv_off .. conv_off
// + C of `proj`) it has seen, for a caller whose own kernel made the convolution.
LRM_API int lrm_conv_tail_update(const void* proj, int dtype, long long stride, int conv_off, int C, int n,
                                 float* tails, const int* cu_seqlens, const int* slots, int seqs,
                                 cudaStream_t stream) {
  if (seqs <= 0 || n <= 1) return 0;
  if (C <= 0 || seqs > 65535 || tails == nullptr) return LRM_BAD_ARGUMENT;
  const dim3 tail_grid((C + 255) / 256, seqs);
  if (dtype == LRM_F32)
    LRM_LAUNCH(conv_tail_update_kernel<float>, tail_grid, 256, 0, stream, static_cast<const float*>(proj), stride,
               conv_off, C, n, tails, cu_seqlens, slots);
  else if (dtype == LRM_BF16)
    LRM_LAUNCH(conv_tail_update_kernel<__nv_bfloat16>, tail_grid, 256, 0, stream,
               static_cast<const __nv_bfloat16*>(proj), stride, conv_off, C, n, tails, cu_seqlens, slots);
  else
    return LRM_BAD_ARGUMENT;
  return 0;
}

// `a` float32 is read at a[t * a_stride + h * d + i].
LRM_API int lrm_delta_prepare(const void* proj, int dtype, long long stride, int conv_off, int b_off,
                              const float* a, long long a_stride, const float* dt_bias, const float* rate, const float* taps, int n,
                              float* tails, const int* cu_seqlens, const int* seq_of_token, const int* slots,
                              float* qf, float* kf, float* vf, float* gf, float* bf, int tokens, int seqs, int H,
                              int G, int d, int dv, float unit_eps, float q_scale, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || d <= 0 || dv <= 0 || n <= 0 || seqs <= 0 || seqs > 65535) return LRM_BAD_ARGUMENT;
  const int threads = 128;
  if (d > 8 * threads || 2 * G + 2 * H + 1 > 65535) return LRM_UNSUPPORTED;
  const int C = 2 * G * d + H * dv;
  const dim3 grid(tokens, 2 * G + 2 * H + 1);
  const dim3 tail_grid((C + 255) / 256, seqs);
  if (dtype == LRM_F32) {
    const float* p = static_cast<const float*>(proj);
    LRM_LAUNCH(delta_prepare_kernel<float>, grid, threads, 0, stream, p, stride, conv_off, b_off, a, a_stride, dt_bias,
               rate, taps, n, static_cast<const float*>(tails), cu_seqlens, seq_of_token, slots, qf, kf, vf, gf, bf, H, G,
               d, dv, unit_eps, q_scale);
    if (n > 1)
      LRM_LAUNCH(conv_tail_update_kernel<float>, tail_grid, 256, 0, stream, p, stride, conv_off, C, n, tails,
                 cu_seqlens, slots);
  } else if (dtype == LRM_BF16) {
    const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(proj);
    LRM_LAUNCH(delta_prepare_kernel<__nv_bfloat16>, grid, threads, 0, stream, p, stride, conv_off, b_off, a,
               a_stride, dt_bias, rate, taps, n, static_cast<const float*>(tails), cu_seqlens, seq_of_token, slots, qf, kf,
               vf, gf, bf, H, G, d, dv, unit_eps, q_scale);
    if (n > 1)
      LRM_LAUNCH(conv_tail_update_kernel<__nv_bfloat16>, tail_grid, 256, 0, stream, p, stride, conv_off, C, n,
                 tails, cu_seqlens, slots);
  } else {
    return LRM_BAD_ARGUMENT;
  }
  return 0;
}
