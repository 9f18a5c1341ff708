// What the kernels of gated softmax attention share (attention_gated.cu, attention_gated_umma.cu): the form of a
// layer's attention, which keys a query sees and in which tiles they lie, and the way from q . k to a score.
#pragma once
#include "common.cuh"

namespace {

constexpr float kLog2e = 1.4426950408889634f;
constexpr int kKeyTile = 64;  // keys per tile (= the cache's page size)

struct Form {
  float scale, cap;            // cap <= 0: none
  int window, keep;            // see first_visible_key; keep: first keys visible to everyone behind them
  const float* sinks;          // [q_heads] or null
  const float* gate;           // null, or pre-activations: gate[t * gate_stride + (per head ? h : h * dv + j)]
  long long gate_stride;
  int gate_per_head;
  void* out;
  long long out_stride;
  float out_scale;
};

__device__ __forceinline__ float gate_at(const Form& f, size_t t, int h, int dv, int j) {
  if (f.gate == nullptr) return f.out_scale;
  const float z = f.gate[t * f.gate_stride + (f.gate_per_head ? h : h * dv + j)];
  return f.out_scale / (1.0f + expf(-z));
}

__device__ __forceinline__ bool sees(const Form& f, int key, int query, int first) {
  return key <= query && (key >= first || key < f.keep);
}

// The tiles a range of queries visits: those of the kept keys that lie before the window's, then the window's.
struct Tiles {
  int kept, first, count;
  __device__ __forceinline__ Tiles(int first_key, int last_key, int keep) : first(first_key / kKeyTile) {
    kept = min((keep + kKeyTile - 1) / kKeyTile, first);
    count = kept + last_key / kKeyTile - first + 1;
  }
  __device__ __forceinline__ int at(int i) const { return i < kept ? i : first + i - kept; }
};

__device__ __forceinline__ float unit_exp2(float x) {  // 2^x on the special-function unit
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float unit_rcp(float x) {  // 1 / x likewise, 0 for infinity
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ float unit_sigmoid(float z) { return unit_rcp(1.0f + unit_exp2(-kLog2e * z)); }

// From q . k to the capped score in the log2 domain: tanh(x) = 1 - 2 / (1 + e^2x), whose error is a rounding
// of the cap wherever x lies. Without a cap a product. Both rise with q . k (where the scale is positive).
struct ScoreMap {
  float mul, cap_log2;
  bool capped;
  __device__ __forceinline__ explicit ScoreMap(const Form& f)
      : mul(f.cap > 0.f ? 2.f * f.scale / f.cap * kLog2e : f.scale * kLog2e), cap_log2(f.cap * kLog2e), capped(f.cap > 0.f) {}
  __device__ __forceinline__ float plain(float dot) const { return dot * mul; }
  __device__ __forceinline__ float cap(float dot) const {
    return fmaf(-2.f * cap_log2, unit_rcp(1.0f + unit_exp2(dot * mul)), cap_log2);
  }
};

inline bool bad_form(const Form& f, int q_heads, int kv_heads, int d, int dv) {
  return q_heads <= 0 || kv_heads <= 0 || q_heads % kv_heads != 0 || d <= 0 || dv <= 0 || f.keep < 0 || f.out == nullptr ||
         f.out_stride < static_cast<long long>(q_heads) * dv ||
         (f.gate != nullptr && f.gate_stride < (f.gate_per_head ? q_heads : static_cast<long long>(q_heads) * dv));
}

inline Form make_form(float scale, float cap, int window, int keep, const float* sinks, const float* gate,
                      long long gate_stride, int gate_per_head, void* out, long long out_stride, float out_scale) {
  // without a window or a chunk every earlier key is visible: kept keys say nothing
  return Form{scale, cap, window, window == 0 ? 0 : keep, sinks, gate, gate_stride, gate_per_head, out, out_stride, out_scale};
}

}  // namespace
