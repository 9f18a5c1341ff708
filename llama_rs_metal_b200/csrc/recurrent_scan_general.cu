// The generalized delta rule and the scan with a bonus for the current token (see recurrent_scan.cuh).
#include "recurrent_scan.cuh"

// The generalized delta rule: q, k, v, g as above (one key head per head), look and put float32
// [T, H, d]: S <- diag(g) S + put (look^T S) + k v^T with both terms reading the old S; o = S^T q.
LRM_API int lrm_general_delta_scan(const float* q, const float* k, const float* v, const float* g, const float* look,
                                   const float* put, float* state, float* out, const int* cu_seqlens,
                                   const int* slots, int seqs, int H, int d, int dv, int tokens, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (H <= 0 || d <= 0 || dv <= 0 || seqs > 65535 || H > 65535) return LRM_BAD_ARGUMENT;
  if (g == nullptr || look == nullptr || put == nullptr) return LRM_BAD_ARGUMENT;
  if (d > 2048) return LRM_UNSUPPORTED;
  return dispatch_scan<3>(q, k, v, g, nullptr, nullptr, look, put, state, out, cu_seqlens, slots, seqs, H, H, d, dv,
                          stream, Rows{tokens});
}

// The read-out before the write, with a bonus for the current token: q, k at [t * q_stride + h * d], v at
// [t * v_stride + h * dv] (strides in floats; columns of a wider activation), g float32 [T, H, d], bonus
// float32 [H, d]: o = (S + diag(bonus) k v^T)^T q, then S <- diag(g) S + k v^T. out float32 [T, H, dv].
LRM_API int lrm_bonus_state_scan(const float* q, const float* k, long long q_stride, const float* v,
                                 long long v_stride, const float* g, const float* bonus, float* state, float* out,
                                 const int* cu_seqlens, const int* slots, int seqs, int H, int d, int dv,
                                 int tokens, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (H <= 0 || d <= 0 || dv <= 0 || seqs > 65535 || H > 65535) return LRM_BAD_ARGUMENT;
  if (g == nullptr || bonus == nullptr || q_stride < static_cast<long long>(H) * d || v_stride < static_cast<long long>(H) * dv)
    return LRM_BAD_ARGUMENT;
  if (d > 2048) return LRM_UNSUPPORTED;
  return dispatch_scan<4>(q, k, v, g, nullptr, nullptr, bonus, nullptr, state, out, cu_seqlens, slots, seqs, H, H, d,
                          dv, stream, Rows{tokens, q_stride, v_stride});
}
