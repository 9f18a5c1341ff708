// Mixers with a fixed-size state per sequence and head: a matrix S [d, dv] in float32 that every
// token updates and reads,
//
//   plain decay (retention):   S <- a S + k v^T                      o = S^T q
//   decay per token:           S <- a_t S + k v^T                    o = S^T q
//   gated delta rule:          S <- diag(g) S;  u = b (v - S^T k);   S <- S + k u^T;   o = S^T q
//   delta rule, head decay:    S <- a_t S;  u = b (v - S^T k);   S <- S + k u^T;   o = S^T q
//   generalized delta rule:    S <- diag(g) S + e (c^T S) + k v^T   (both terms read the old S)   o = S^T q
//   bonus for the newest:      o = (S + diag(m) k v^T)^T q;   S <- diag(g) S + k v^T   (read before the write)
//
// with a one decay per head (or, per token, one per head and token: state-space and matrix-memory
// mixers, whose step size or input gate the caller has multiplied into v), g one decay per head
// and key channel and token, b one step size per head and token; in the generalized rule c is the
// direction that is read (a unit key) and e what is written back along it (minus a removal rate
// per key channel times that direction), both per head, key channel and token; m is one factor per
// head and key channel that the current token's own contribution has in the read-out. Everything here is float32: the inputs are prepared in float32 by the kernels
// below (rotation, short convolutions, unit norms, decays), the state lives in float32 in the
// cache's state storage, one matrix per slot and head, and is carried from step to step.
//
// The scan: one CTA per (sequence, head, tile of value columns). Columns of S do not depend on
// one another, so a CTA keeps its columns in registers for the whole step: thread (column j,
// part p of P) holds a run of consecutive rows of column j. Per token every thread forms, over its
// rows, the partial sums  r = sum g_i S_ij k_i  (delta rules)  and  s = sum g_i S_ij q_i, which are added
// over the P parts by shuffles, and with  c = sum k_i q_i, which is the same for all columns and made once
// per stage,
//   u_j = b (v_j - r)   (or v_j without the delta rule),   o_j = s + u_j c,   S_ij <- g_i S_ij + k_i u_j,
// which is the update above with the read-out taken after the write. Only r is waited for before the next
// token: the sums s of four tokens are added over the parts together. Tokens are staged through
// shared memory a chunk at a time by asynchronous copies, the next chunk under way while this
// one is worked on, so the inner loop has no block-wide barrier and waits for no load. A step of one
// token (decoding) and a step of a whole prompt run the same arithmetic in the same order, so
// the state after a prompt does not depend on how it was cut.
//
// A sequence of padding (slot < 0) starts from zero and stores nothing.
//
// The scan's kernels; each mode is built in a source file of its own kind (recurrent_scan.cu and
// recurrent_scan_*.cu).
#pragma once
#include "common.cuh"

extern int g_scan_rows;  // most rows a thread holds (tuning: lrm_linear_state_scan_rows); recurrent_scan.cu

namespace {

constexpr int kScanThreads = 128;
constexpr int kChunk = 16;  // tokens per stage, halved while two stages do not fit the shared memory

__device__ __forceinline__ void scan_cp_async(float* dst, const float* src, bool valid, bool wide) {
  const uint32_t d = static_cast<uint32_t>(__cvta_generic_to_shared(dst));
  if (wide)
    asm volatile("cp.async.ca.shared.global [%0], [%1], 16, %2;\n" ::"r"(d), "l"(src), "r"(valid ? 16 : 0));
  else
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"(d), "l"(src), "r"(valid ? 4 : 0));
}

// Thread (column j, part p) holds rows p * ROWS .. p * ROWS + ROWS - 1 of column j. A token's q, k
// and g rows lie in shared memory as [P][ROWS + 4] (the 4 floats between the parts keep the parts'
// 16-byte reads on different banks); tokens come in chunks of kChunk, two chunks in flight.
// MODE 0: one decay per head (head_decay); 1: the gated delta rule (g, beta); 2: one decay per head
// and token (in `beta`'s place, [T, H]); 3: the generalized delta rule (g, and the two more rows
// `look` = c and `put` = e per token, [T, H, d]): with t_j = sum_i c_i S_ij over the old state,
// S_ij <- g_i S_ij + e_i t_j + k_i v_j and o_j = sum_i g_i S_ij q_i + t_j (e . q) + v_j (k . q);
// 4: the read-out before the write with a bonus (g, and `look` = m [H, d], the same for every token):
// o_j = sum_i S_ij q_i + v_j sum_i m_i k_i q_i, then S_ij <- g_i S_ij + k_i v_j: nothing a token adds to
// the state waits for a sum over it; 5: the delta rule with one decay per head and token (`beta`
// [T, H] step sizes, `put` [T, H] decays).
// q and k rows of a token are q_stride floats after those of the token before, v rows v_stride.
template <int ROWS, int MODE, int PT>
__global__ __launch_bounds__(kScanThreads) void linear_scan_kernel(
    const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v,
    const float* __restrict__ g, const float* __restrict__ head_decay, const float* __restrict__ beta,
    const float* __restrict__ look, const float* __restrict__ put,
    float* __restrict__ state, float* __restrict__ out, const int* __restrict__ cu_seqlens,
    const int* __restrict__ slots, int H, int KH, int d, int dv, int P_any, int chunk, long long q_stride,
    long long v_stride, int wide_rows) {
  extern __shared__ __align__(16) float smem[];
  constexpr bool DELTA = MODE == 1 || MODE == 5;
  constexpr bool GEN = MODE == 3;
  constexpr bool BONUS = MODE == 4;
  constexpr bool ROW_DECAY = MODE == 1 || MODE == 3 || MODE == 4;  // a row g of decays per token
  constexpr int NR = GEN ? 5 : ROW_DECAY ? 3 : 2;      // rows of d floats a token brings
  constexpr int RS = ROWS + 4;
  const int P = PT > 0 ? PT : P_any;                    // known to the compiler where that pays
  const int TS = P * RS, COLS = kScanThreads / P;
  const int VS = (COLS + 3) & ~3;                       // v of a token, padded to whole 16 bytes
  const int TOKEN = NR * TS + VS + 4;                   // q | k | (g) | (look | put) | v | beta, decay, dot, dot
  const int STAGE = chunk * TOKEN;

  const int tid = threadIdx.x, pidx = tid % P, jl = tid / P;
  const int h = blockIdx.y, b = blockIdx.z, kh = h / (H / KH);
  const int j = blockIdx.x * COLS + jl;
  pdl_wait();
  const int start = cu_seqlens[b], n = cu_seqlens[b + 1] - start;
  const int slot = slots[b];
  float S[ROWS];
  float* mine = slot >= 0 ? state + (static_cast<size_t>(slot) * H + h) * d * dv : nullptr;
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int row = pidx * ROWS + i;
    S[i] = (mine != nullptr && row < d && j < dv) ? mine[static_cast<size_t>(row) * dv + j] : 0.f;
  }
  const float a = MODE == 0 ? head_decay[h] : 1.f;
  float* factors = smem + 2 * STAGE;  // BONUS: the head's factors, laid out like a token's row
  if constexpr (BONUS)
    for (int r = tid; r < ROWS * P; r += kScanThreads) factors[(r / ROWS) * RS + r % ROWS] = r < d ? look[h * d + r] : 0.f;
  // 16-byte copies where every row of the inputs starts on a 16-byte boundary
  const bool wide = wide_rows && COLS % 4 == 0;
  const int step = wide ? 4 : 1;

  auto issue = [&](int c0, int stage) {
    float* base = smem + stage * STAGE;
    const int cn = min(chunk, n - c0);
    const int per_token = ROWS * P / step;  // granules of a q (k, g) row, padding rows included
    for (int idx = tid; idx < cn * per_token; idx += kScanThreads) {
      const int c = idx / per_token, r = (idx % per_token) * step;
      const size_t tok = static_cast<size_t>(start + c0 + c);
      const bool in = r < d;
      float* dst = base + c * TOKEN + (r / ROWS) * RS + r % ROWS;
      scan_cp_async(dst, q + tok * q_stride + kh * d + (in ? r : 0), in, wide);
      scan_cp_async(dst + TS, k + tok * q_stride + kh * d + (in ? r : 0), in, wide);
      if (ROW_DECAY) scan_cp_async(dst + 2 * TS, g + (tok * H + h) * d + (in ? r : 0), in, wide);
      if (GEN) {
        scan_cp_async(dst + 3 * TS, look + (tok * H + h) * d + (in ? r : 0), in, wide);
        scan_cp_async(dst + 4 * TS, put + (tok * H + h) * d + (in ? r : 0), in, wide);
      }
    }
    const int v_per_token = COLS / step;
    for (int idx = tid; idx < cn * v_per_token; idx += kScanThreads) {
      const int c = idx / v_per_token, cl = (idx % v_per_token) * step, col = blockIdx.x * COLS + cl;
      const size_t tok = static_cast<size_t>(start + c0 + c);
      const bool in = col < dv;
      scan_cp_async(base + c * TOKEN + NR * TS + cl, v + tok * v_stride + h * dv + (in ? col : 0), in, wide);
    }
    if (MODE == 1 || MODE == 2 || MODE == 5)
      for (int c = tid; c < cn; c += kScanThreads) {
        scan_cp_async(base + c * TOKEN + NR * TS + VS, beta + static_cast<size_t>(start + c0 + c) * H + h,
                      true, false);
        if (MODE == 5)
          scan_cp_async(base + c * TOKEN + NR * TS + VS + 1, put + static_cast<size_t>(start + c0 + c) * H + h,
                        true, false);
      }
    asm volatile("cp.async.commit_group;\n" ::);
  };

  if (n > 0) issue(0, 0);
  for (int c0 = 0, it = 0; c0 < n; c0 += chunk, ++it) {
    const int cn = min(chunk, n - c0);
    if (c0 + chunk < n) {
      issue(c0 + chunk, (it + 1) & 1);
      asm volatile("cp.async.wait_group 1;\n" ::);
    } else {
      asm volatile("cp.async.wait_group 0;\n" ::);
    }
    __syncthreads();
    float* base = smem + (it & 1) * STAGE;
    // What the read-out needs of a token beside the state is the same for all columns: k . q (under the
    // factors of a bonus), and e . q. Eight lanes per token make it once per stage.
    for (int c = tid >> 3; c < cn; c += kScanThreads / 8) {
      float* token = base + c * TOKEN;
      float kq = 0.f, eq = 0.f;
      for (int r = (tid & 7) * 4; r < ROWS * P; r += 32) {
        const int at = (r / ROWS) * RS + r % ROWS;
        const float4 q4 = *reinterpret_cast<const float4*>(token + at);
        float4 k4 = *reinterpret_cast<const float4*>(token + TS + at);
        if constexpr (BONUS) {
          const float4 f4 = *reinterpret_cast<const float4*>(factors + at);
          k4.x *= f4.x, k4.y *= f4.y, k4.z *= f4.z, k4.w *= f4.w;
        }
        kq = fmaf(k4.x, q4.x, fmaf(k4.y, q4.y, fmaf(k4.z, q4.z, fmaf(k4.w, q4.w, kq))));
        if constexpr (GEN) {
          const float4 e4 = *reinterpret_cast<const float4*>(token + 4 * TS + at);
          eq = fmaf(e4.x, q4.x, fmaf(e4.y, q4.y, fmaf(e4.z, q4.z, fmaf(e4.w, q4.w, eq))));
        }
      }
      const unsigned lanes = 0xffu << (tid & 24);
#pragma unroll
      for (int o = 1; o < 8; o <<= 1) {
        kq += __shfl_xor_sync(lanes, kq, o);
        if (GEN) eq += __shfl_xor_sync(lanes, eq, o);
      }
      if ((tid & 7) == 0) {
        token[NR * TS + VS + 2] = kq;
        if (GEN) token[NR * TS + VS + 3] = eq;
      }
    }
    __syncthreads();
    // What a token brings to this thread, in registers.
    struct Brought {
      float4 q[ROWS / 4], k[ROWS / 4], g[ROW_DECAY ? ROWS / 4 : 1], c[GEN ? ROWS / 4 : 1], e[GEN ? ROWS / 4 : 1];
      float v;
      float4 scalars;
    };
    auto fetch = [&](int c, Brought& t) {
      const float* token = base + c * TOKEN;
      const float* qc = token + pidx * RS;
#pragma unroll
      for (int i = 0; i < ROWS / 4; ++i) {
        t.q[i] = *reinterpret_cast<const float4*>(qc + 4 * i);
        t.k[i] = *reinterpret_cast<const float4*>(qc + TS + 4 * i);
        if constexpr (ROW_DECAY) t.g[i] = *reinterpret_cast<const float4*>(qc + 2 * TS + 4 * i);
        if constexpr (GEN) {
          t.c[i] = *reinterpret_cast<const float4*>(qc + 3 * TS + 4 * i);
          t.e[i] = *reinterpret_cast<const float4*>(qc + 4 * TS + 4 * i);
        }
      }
      t.v = token[NR * TS + jl];
      t.scalars = *reinterpret_cast<const float4*>(token + NR * TS + VS);
    };
    // One token: the state moves on; -> this thread's share of the read-out and what every part adds to it.
    auto advance = [&](const Brought& t, float& share, float& whole) {
      const float at = MODE == 2 ? t.scalars.x : MODE == 5 ? t.scalars.y : a;
      float r0 = 0.f, r1 = 0.f, s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int n4 = 0; n4 < ROWS / 4; ++n4) {
        const int i = 4 * n4;
        const float4 k4 = t.k[n4], q4 = t.q[n4];
        float4 g4 = make_float4(at, at, at, at);
        if constexpr (ROW_DECAY) g4 = t.g[n4];
        if constexpr (GEN) {  // what the old state holds along `look`, before the decay
          const float4 c4 = t.c[n4];
          r0 = fmaf(S[i], c4.x, r0), r1 = fmaf(S[i + 1], c4.y, r1);
          r0 = fmaf(S[i + 2], c4.z, r0), r1 = fmaf(S[i + 3], c4.w, r1);
        }
        if constexpr (BONUS) {  // the old state is read, then decayed
          s0 = fmaf(S[i], q4.x, s0), s1 = fmaf(S[i + 1], q4.y, s1);
          s0 = fmaf(S[i + 2], q4.z, s0), s1 = fmaf(S[i + 3], q4.w, s1);
        }
        S[i] *= g4.x, S[i + 1] *= g4.y, S[i + 2] *= g4.z, S[i + 3] *= g4.w;
        if (DELTA) {
          r0 = fmaf(S[i], k4.x, r0), r1 = fmaf(S[i + 1], k4.y, r1);
          r0 = fmaf(S[i + 2], k4.z, r0), r1 = fmaf(S[i + 3], k4.w, r1);
        }
        if constexpr (!BONUS) {
          s0 = fmaf(S[i], q4.x, s0), s1 = fmaf(S[i + 1], q4.y, s1);
          s0 = fmaf(S[i + 2], q4.z, s0), s1 = fmaf(S[i + 3], q4.w, s1);
        }
      }
      float r = r0 + r1;
      if (DELTA || GEN) {
#pragma unroll
        for (int o = P >> 1; o > 0; o >>= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
      }
      const float u = DELTA ? t.scalars.x * (t.v - r) : t.v;
#pragma unroll
      for (int n4 = 0; n4 < ROWS / 4; ++n4) {
        const int i = 4 * n4;
        S[i] = fmaf(t.k[n4].x, u, S[i]), S[i + 1] = fmaf(t.k[n4].y, u, S[i + 1]);
        S[i + 2] = fmaf(t.k[n4].z, u, S[i + 2]), S[i + 3] = fmaf(t.k[n4].w, u, S[i + 3]);
        if constexpr (GEN) {
          S[i] = fmaf(t.e[n4].x, r, S[i]), S[i + 1] = fmaf(t.e[n4].y, r, S[i + 1]);
          S[i + 2] = fmaf(t.e[n4].z, r, S[i + 2]), S[i + 3] = fmaf(t.e[n4].w, r, S[i + 3]);
        }
      }
      share = s0 + s1;
      whole = u * t.scalars.z;
      if constexpr (GEN) whole = fmaf(r, t.scalars.w, whole);
    };
    float* out_row = out + (static_cast<size_t>(start + c0) * H + h) * dv + j;
    const size_t out_step = static_cast<size_t>(H) * dv;
    int c = 0;
    if constexpr (PT >= 4) {
      // Four tokens at a time: their read-outs are added over the parts together, every exchange halving
      // the tokens a thread still holds (6 exchanges and fewer instead of 4 log2(P)); the thread that
      // ends with a token's sum writes it. The tree of additions is the one of a single token.
      for (; c + 4 <= cn; c += 4) {
        float s[4], w[4];
        Brought now, next;
        if constexpr (DELTA || GEN) {  // bound by the chain through the sums over the state: no room to look ahead
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            fetch(c + e, now);
            advance(now, s[e], w[e]);
          }
        } else {
          fetch(c, now);
#pragma unroll
          for (int e = 0; e < 4; ++e) {  // the next token's rows are on their way while this one is worked on
            if (e < 3) fetch(c + e + 1, e & 1 ? now : next);
            advance(e & 1 ? next : now, s[e], w[e]);
          }
        }
        const bool high = (pidx & (PT / 2)) != 0, odd = (pidx & (PT / 4)) != 0;
        const float give0 = high ? s[0] : s[2], give1 = high ? s[1] : s[3];
        const float a0 = (high ? s[2] : s[0]) + __shfl_xor_sync(0xffffffffu, give0, PT / 2);
        const float a1 = (high ? s[3] : s[1]) + __shfl_xor_sync(0xffffffffu, give1, PT / 2);
        float x = (odd ? a1 : a0) + __shfl_xor_sync(0xffffffffu, odd ? a0 : a1, PT / 4);
#pragma unroll
        for (int o = PT / 8; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
        if ((pidx & (PT / 4 - 1)) == 0 && j < dv)
          out_row[(c + (high ? 2 : 0) + (odd ? 1 : 0)) * out_step] = x + (high ? (odd ? w[3] : w[2]) : (odd ? w[1] : w[0]));
      }
    }
    for (; c < cn; ++c) {
      float s, w;
      Brought now;
      fetch(c, now);
      advance(now, s, w);
#pragma unroll
      for (int o = P >> 1; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if (pidx == 0 && j < dv) out_row[c * out_step] = s + w;
    }
    __syncthreads();
  }
  if (mine != nullptr) {
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int row = pidx * ROWS + i;
      if (row < d && j < dv) mine[static_cast<size_t>(row) * dv + j] = S[i];
    }
  }
}

// How far apart a token's q and k rows, and its v row, are from those of the token before (0: packed), and
// how many tokens the step has.
struct Rows {
  int tokens;
  long long q = 0, v = 0;
};

constexpr int kLongWalk = 16;  // tokens per sequence from which a scan is a long walk

template <int ROWS, int MODE, int PT>
int launch_scan(const float* q, const float* k, const float* v, const float* g, const float* head_decay,
                const float* beta, const float* look, const float* put, float* state, float* out, const int* cu_seqlens, const int* slots,
                int seqs, int H, int KH, int d, int dv, int P, const Rows& rows, cudaStream_t stream) {
  constexpr int NR = MODE == 3 ? 5 : MODE == 1 || MODE == 4 ? 3 : 2;
  const int COLS = kScanThreads / P, TS = P * (ROWS + 4), VS = (COLS + 3) & ~3;
  int chunk = kChunk;
  while (chunk > 1 && sizeof(float) * 2 * chunk * (static_cast<size_t>(NR) * TS + VS + 4) > 200 * 1024) chunk >>= 1;
  const size_t bytes = sizeof(float) * (2 * chunk * (static_cast<size_t>(NR) * TS + VS + 4) + (MODE == 4 ? TS : 0));
  if (bytes > 200 * 1024) return LRM_UNSUPPORTED;
  static bool raised = false;  // per instantiation
  if (bytes > 48 * 1024 && !raised) {
    cudaError_t e = cudaFuncSetAttribute(linear_scan_kernel<ROWS, MODE, PT>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    raised = true;
  }
  const long long q_stride = rows.q > 0 ? rows.q : static_cast<long long>(KH) * d;
  const long long v_stride = rows.v > 0 ? rows.v : static_cast<long long>(H) * dv;
  auto aligned = [](const float* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const int wide = d % 4 == 0 && dv % 4 == 0 && q_stride % 4 == 0 && v_stride % 4 == 0 && aligned(q) && aligned(k) &&
                   aligned(v) && aligned(g) && (MODE != 3 || (aligned(look) && aligned(put)));
  const dim3 grid((dv + COLS - 1) / COLS, H, seqs);
  // A long walk is bound by its tokens' latency and wants an SM to itself. Let in while the kernel before
  // still runs, its CTAs pile up on the SMs that kernel leaves first (one prompt of 2,048 tokens: 800
  // us in the middle of a step against 260 alone), so it starts when that kernel is done.
  const int pdl = g_lrm_pdl;
  if (rows.tokens >= static_cast<long long>(seqs) * kLongWalk) g_lrm_pdl = 0;
  const cudaError_t launched = lrm_launch(linear_scan_kernel<ROWS, MODE, PT>, grid, kScanThreads, bytes, stream, q, k, v, g,
                                          head_decay, beta, look, put, state, out, cu_seqlens, slots, H, KH, d, dv, P,
                                          chunk, q_stride, v_stride, wide);
  g_lrm_pdl = pdl;
  if (launched != cudaSuccess) return static_cast<int>(launched);
  return 0;
}

// How a head's key rows are cut over threads: P parts (a power of two up to 32) of ROWS rows.
// Few parts when the head is small (less to add up by shuffles), more when it is large (the
// registers a thread can keep bound ROWS to 64).
inline void scan_shape(int d, int* rows, int* parts, int most_rows) {
  int P = 1;
  while (P < 32 && (d + P - 1) / P > most_rows) P <<= 1;
  int need = (d + P - 1) / P, R = 4;
  while (R < need) R <<= 1;
  *rows = R;
  *parts = P;
}

template <int MODE>
int dispatch_scan(const float* q, const float* k, const float* v, const float* g, const float* head_decay,
                  const float* beta, const float* look, const float* put, float* state, float* out, const int* cu_seqlens, const int* slots,
                  int seqs, int H, int KH, int d, int dv, cudaStream_t stream, const Rows& rows) {
  int R, P;
  scan_shape(d, &R, &P, g_scan_rows);
  if (g_scan_rows > 8) {
    // Few sequences (one prompt) can leave most SMs without a CTA, and every CTA walks its tokens one
    // after another: with half the rows per thread a head's columns go to twice as many CTAs and a
    // token's chain of sums is shorter (one prompt of 2,048 tokens: 8 heads of 128 x 128 with a plain
    // decay 260 against 323 us). Steps that fill half the device keep the standard shape.
    const long long ctas = static_cast<long long>((dv + kScanThreads / P - 1) / (kScanThreads / P)) * H * seqs;
    if (2 * ctas <= 148) scan_shape(d, &R, &P, g_scan_rows / 2);
  }
#define LRM_SCAN(N, PARTS)                                                                            \
  return launch_scan<N, MODE, PARTS>(q, k, v, g, head_decay, beta, look, put, state, out, cu_seqlens, slots, seqs, H, \
                                     KH, d, dv, P, rows, stream)
  // heads of up to 256 at the usual shapes: the number of parts is known, so the sums over the parts are
  // straight code and a token's work overlaps its neighbours'
  if (R == 16 && P == 4) LRM_SCAN(16, 4);
  if (R == 16 && P == 8) LRM_SCAN(16, 8);
  if (R == 16 && P == 16) LRM_SCAN(16, 16);
  if (R == 8 && P == 8) LRM_SCAN(8, 8);
  if (R == 8 && P == 16) LRM_SCAN(8, 16);
  switch (R) {
    case 4: LRM_SCAN(4, 0);
    case 8: LRM_SCAN(8, 0);
    case 16: LRM_SCAN(16, 0);
    case 32: LRM_SCAN(32, 0);
    case 64: LRM_SCAN(64, 0);
  }
#undef LRM_SCAN
  return LRM_UNSUPPORTED;
}

}  // namespace
