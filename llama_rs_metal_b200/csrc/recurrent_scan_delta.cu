// The gated delta rule with a decay per key channel, and with one decay per head (see recurrent_scan.cuh).
#include "recurrent_scan.cuh"

// Called by lrm_linear_state_scan, which has checked the arguments.
extern "C" int lrm_scan_gated_delta(const float* q, const float* k, const float* v, const float* g, const float* beta,
                                    float* state, float* out, const int* cu_seqlens, const int* slots, int seqs, int H,
                                    int KH, int d, int dv, int tokens, cudaStream_t stream) {
  return dispatch_scan<1>(q, k, v, g, nullptr, beta, nullptr, nullptr, state, out, cu_seqlens, slots, seqs, H, KH, d, dv,
                          stream, Rows{tokens});
}

// The delta rule with one decay per head and token: q, k float32 [T, KH, d], v [T, H, dv], decay and beta
// float32 [T, H]: S <- decay S;  S <- S + k (beta (v - S^T k))^T;  o = S^T q.
LRM_API int lrm_head_decay_delta_scan(const float* q, const float* k, const float* v, const float* decay,
                                      const float* beta, float* state, float* out, const int* cu_seqlens,
                                      const int* slots, int seqs, int H, int KH, int d, int dv, int tokens, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (H <= 0 || KH <= 0 || H % KH || d <= 0 || dv <= 0 || seqs > 65535 || H > 65535) return LRM_BAD_ARGUMENT;
  if (decay == nullptr || beta == nullptr) return LRM_BAD_ARGUMENT;
  if (d > 2048) return LRM_UNSUPPORTED;
  return dispatch_scan<5>(q, k, v, nullptr, nullptr, beta, nullptr, decay, state, out, cu_seqlens, slots, seqs, H, KH, d,
                          dv, stream, Rows{tokens});
}
