// Causal grouped-query attention without a softmax: the weight of a visible key is
//   sigmoid(scale * (q . k) + offset_h),
// one offset per query head, and nothing is normalized over the keys:
//   out = sum_p w_p v_p  [* sigmoid(gate)] * out_scale,
// with an optional gate per head and value dimension (pre-activations in float32, read where the result
// leaves the kernel). Scores, weights, sums and the gate are float32. Because a key's share does not
// depend on the other keys there is no running maximum, no mass, and partial results of any split of
// the keys simply add up. A window w > 0 shows the query at position p the keys p - w + 1 .. p, a
// negative one the chunk of -w positions it stands in (first_visible_key), 0 every earlier key.
// The result of token t, head h goes to out[t * out_stride + h * dv]: a column range of a wider row.
//
//  * row-wise: one warp per (query, head), keys one at a time in ascending order, from the step's
//    packed keys or the paged cache, both dtypes, head sizes up to 1024: the attention of the float32
//    path, and of sizes the tiled kernels refuse.
//  * tiled (bfloat16, head size 32, 64, 96 or 128, values as wide as keys): 64 queries of one head per
//    CTA over 64-key tiles on mma.sync, double buffered by cp.async, from packed keys (prompts) or
//    the cache's pages (portions).
//  * decode (same sizes): one query per sequence over the cache; the CTAs of a thread-block cluster
//    take runs of a sequence's pages, add their sums through distributed shared memory in rank
//    order, and each writes a share of the columns: one launch, no partial rows in memory.
// Rows of a tile outside the visible range are zero-filled on the way into shared memory, so stale
// cache contents never reach a product.
#include <cooperative_groups.h>

#include "attention_mma.cuh"

namespace {

namespace cg = cooperative_groups;

constexpr float kLog2e = 1.4426950408889634f;

struct Output {
  void* out;
  long long stride;         // elements between two tokens' rows
  const float* gate;        // pre-activations: gate[t * gate_stride + h * dv + j], or null
  long long gate_stride;
  float scale;              // factor on the result
};

__device__ __forceinline__ float gated(float v, const float* gate, size_t at, float scale) {
  if (gate != nullptr) v *= 1.0f / (1.0f + expf(-gate[at]));
  return v * scale;
}

// --------------------------------------------------------------------------- row-wise
template <typename A, int PER, bool PAGED>
__global__ void sigmoid_rowwise_kernel(const A* q, const A* k, const A* v, Output o, const int* __restrict__ cu_seqlens,
                                       const int* __restrict__ seq_of_token, const int* __restrict__ positions,
                                       const int* __restrict__ page_table, int table_stride,
                                       const int* __restrict__ slots, const int* __restrict__ kv_lens, int q_heads,
                                       int kv_heads, int d, int dv, int page_size, float scale, int window,
                                       const float* __restrict__ offset) {
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, kh = h / (q_heads / kv_heads);
  const int lane = threadIdx.x & 31;
  int pos, start = 0;
  const int* table = nullptr;
  if (PAGED) {
    const int b = seq_of_token != nullptr ? seq_of_token[t] : t;
    pos = positions != nullptr ? positions[t] : kv_lens[b] - 1;
    table = page_table + static_cast<size_t>(slots[b]) * table_stride;
  } else {
    start = cu_seqlens[seq_of_token[t]];
    pos = t - start;
  }
  const A* qr = q + (static_cast<size_t>(t) * q_heads + h) * d;
  const float add = offset[h];
  float qv[PER], acc[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int j = lane + 32 * i;
    qv[i] = j < d ? to_f32(qr[j]) : 0.f;
    acc[i] = 0.f;
  }
  for (int p = first_visible_key(pos, window); p <= pos; ++p) {
    size_t key;  // row number among rows of one key head's width
    if (PAGED) {
      const int page = table[p / page_size];
      key = (static_cast<size_t>(page) * kv_heads + kh) * page_size + p % page_size;
    } else {
      key = static_cast<size_t>(start + p) * kv_heads + kh;
    }
    const A* kr = k + key * d;
    const A* vr = v + key * dv;
    float dot = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int j = lane + 32 * i;
      if (j < d) dot = fmaf(qv[i], to_f32(kr[j]), dot);
    }
    const float s = fmaf(warp_sum(dot), scale, add);
    const float w = 1.0f / (1.0f + expf(-s));
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int j = lane + 32 * i;
      if (j < dv) acc[i] = fmaf(w, to_f32(vr[j]), acc[i]);
    }
  }
  A* dst = static_cast<A*>(o.out) + static_cast<size_t>(t) * o.stride + h * dv;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int j = lane + 32 * i;
    if (j < dv) dst[j] = from_f32<A>(gated(acc[i], o.gate, static_cast<size_t>(t) * o.gate_stride + h * dv + j, o.scale));
  }
}

// --------------------------------------------------------------------------- tiles
__device__ __forceinline__ float rcp_fast(float x) {  // 1 / x on the special-function unit, 0 for infinity
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// sigmoid of a score given as -score * log2(e)
__device__ __forceinline__ float weight_of(float negated_log2) { return rcp_fast(1.0f + exp2_fast(negated_log2)); }

// Rows [lo, hi) of 64 x D elements (row pitch `pitch`) into a padded tile, the others zero-filled.
template <int D>
__device__ __forceinline__ void load_rows(__nv_bfloat16* dst, const __nv_bfloat16* src, size_t pitch, int lo, int hi) {
  constexpr int STRIDE = D + 8, CHUNKS = D / 8;
#pragma unroll 4
  for (int idx = threadIdx.x; idx < kTile * CHUNKS; idx += kThreads) {
    const int r = idx / CHUNKS, c = (idx % CHUNKS) * 8;
    const bool ok = r >= lo && r < hi;
    cp_async16(dst + r * STRIDE + c, ok ? src + r * pitch + c : src, ok ? 16 : 0);
  }
}

// PAGED: the queries are the last n of len tokens and keys come from the cache's pages; otherwise the
// sequence's own packed keys (n == len, queries from position 0).
template <int D, bool PAGED>
__global__ __launch_bounds__(kThreads) void sigmoid_tiled_kernel(
    const __nv_bfloat16* q, const __nv_bfloat16* k, const __nv_bfloat16* v, Output out,
    const int* __restrict__ cu_seqlens, const int* __restrict__ page_table, int table_stride,
    const int* __restrict__ slots, const int* __restrict__ kv_lens, int q_heads, int kv_heads, float scale, int window,
    const float* __restrict__ offset) {
  constexpr int STRIDE = D + 8, TILE = kTile * STRIDE;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(smem_raw);  // [2][64][STRIDE]
  __nv_bfloat16* Vs = Ks + 2 * TILE;

  const int qt = gridDim.z - 1 - blockIdx.z;  // the longest rows of work first
  const int h = blockIdx.x, b = blockIdx.y;
  const int start = cu_seqlens[b], n = cu_seqlens[b + 1] - start;
  const int q0 = qt * kTile;
  if (q0 >= n) return;
  const int len = PAGED ? kv_lens[b] : n, before = len - n;
  const int kh = h / (q_heads / kv_heads);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int row0 = q0 + 16 * warp;  // this warp's first query, counted within the portion
  const int* table = PAGED ? page_table + static_cast<size_t>(slots[b]) * table_stride : nullptr;
  const float negated = -scale * kLog2e, add = -offset[h] * kLog2e;
  pdl_wait();

  uint32_t qa[D / 16][4];
  load_q<D>(qa, q + (static_cast<size_t>(start + row0) * q_heads + h) * D, static_cast<size_t>(q_heads) * D, n - row0);
  float o[D / 8][4];
#pragma unroll
  for (int dn = 0; dn < D / 8; ++dn)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[dn][e] = 0.f;

  const int first_key = first_visible_key(before + q0, window);
  const int kt_first = first_key / kTile, kt_last = (before + min(q0 + kTile, n) - 1) / kTile;
  const int query[2] = {before + row0 + g, before + row0 + g + 8};
  const int row_first[2] = {first_visible_key(query[0], window), first_visible_key(query[1], window)};
  // tiles all of whose keys every query of the CTA sees need no test per score
  const int whole_from = first_visible_key(before + min(q0 + kTile, n) - 1, window), whole_to = before + q0;
  const size_t pitch = PAGED ? D : static_cast<size_t>(kv_heads) * D;
  auto issue = [&](int kt, int stage) {
    const int lo = first_key - kt * kTile;
    int hi = len - kt * kTile;
    size_t base;
    if (PAGED) {
      const int page = table[kt];
      if (page < 0) hi = 0;
      base = (static_cast<size_t>(max(page, 0)) * kv_heads + kh) * kTile * D;
    } else {
      base = (static_cast<size_t>(start + kt * kTile) * kv_heads + kh) * D;
    }
    load_rows<D>(Ks + stage * TILE, k + base, pitch, lo, hi);
    load_rows<D>(Vs + stage * TILE, v + base, pitch, lo, hi);
    cp_async_commit();
  };
  issue(kt_first, 0);
  for (int kt = kt_first; kt <= kt_last; ++kt) {
    const int stage = (kt - kt_first) & 1;
    if (kt < kt_last) {
      issue(kt + 1, stage ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    float s[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[nt][e] = 0.f;
    scores<D, 8>(s, qa, Ks + stage * TILE);
    if (kt * kTile >= whole_from && (kt + 1) * kTile - 1 <= whole_to) {
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[nt][e] = weight_of(fmaf(s[nt][e], negated, add));
    } else {
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int key = kt * kTile + 8 * nt + 2 * t + (e & 1);
          const bool visible = key <= query[e >> 1] && key >= row_first[e >> 1];
          s[nt][e] = visible ? weight_of(fmaf(s[nt][e], negated, add)) : 0.f;
        }
    }
    weighted_values<D, 8>(o, s, Vs + stage * TILE);
    __syncthreads();
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int row = row0 + g + 8 * half;
    if (row >= n) continue;
    const size_t tok = static_cast<size_t>(start + row);
    __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(out.out) + tok * out.stride + h * D;
    const size_t gate_at = tok * out.gate_stride + static_cast<size_t>(h) * D;
#pragma unroll
    for (int dn = 0; dn < D / 8; ++dn) {
      const int c = 8 * dn + 2 * t;
      const float a = gated(o[dn][2 * half], out.gate, gate_at + c, out.scale);
      const float e = gated(o[dn][2 * half + 1], out.gate, gate_at + c + 1, out.scale);
      *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(a, e);
    }
  }
}

// --------------------------------------------------------------------------- decode
// A cluster of gridDim.x CTAs per (sequence, kv head, group of up to 16 query heads) [blockIdx.y]; the
// CTA of rank r takes a run of the visible pages, its four warps 16 keys of every page each.
template <int D>
__global__ __launch_bounds__(kThreads) void sigmoid_decode_kernel(
    const __nv_bfloat16* q, const __nv_bfloat16* k_pages, const __nv_bfloat16* v_pages, Output out,
    const int* __restrict__ page_table, int table_stride, const int* __restrict__ slots,
    const int* __restrict__ kv_lens, int q_heads, int kv_heads, int row_groups, float scale, int window,
    const float* __restrict__ offset) {
  constexpr int STRIDE = D + 8, TILE = kTile * STRIDE;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(smem_raw);
  __nv_bfloat16* Vs = Ks + 2 * TILE;
  const int ranks = gridDim.x, rank = blockIdx.x;
  const int rg = blockIdx.y % row_groups, kh = (blockIdx.y / row_groups) % kv_heads;
  const int b = blockIdx.y / (row_groups * kv_heads);
  const int group = q_heads / kv_heads, head0 = kh * group + 16 * rg;
  const int rows = min(16, group - 16 * rg);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int len = kv_lens[b];
  const int first_key = len > 0 ? first_visible_key(len - 1, window) : 0;
  const int page_first = first_key / kTile, page_end = (len + kTile - 1) / kTile;
  const int per_rank = (page_end - page_first + ranks - 1) / ranks;
  const int p_begin = page_first + rank * per_rank, p_end = min(page_end, p_begin + per_rank);
  const int* table = page_table + static_cast<size_t>(slots[b]) * table_stride;
  const float negated = -scale * kLog2e;
  const float add[2] = {g < rows ? -offset[head0 + g] * kLog2e : 0.f, g + 8 < rows ? -offset[head0 + g + 8] * kLog2e : 0.f};

  auto issue = [&](int page_index, int stage) {
    const size_t base = (static_cast<size_t>(table[page_index]) * kv_heads + kh) * kTile * D;
    load_rows<D>(Ks + stage * TILE, k_pages + base, D, first_key - page_index * kTile, len - page_index * kTile);
    load_rows<D>(Vs + stage * TILE, v_pages + base, D, first_key - page_index * kTile, len - page_index * kTile);
    cp_async_commit();
  };
  // only q and the newest key and value row (in the last page) come from the kernel before this one
  const bool early = p_begin < p_end && p_begin != page_end - 1;
  if (early) issue(p_begin, 0);
  pdl_wait();
  if (!early && p_begin < p_end) issue(p_begin, 0);

  uint32_t qa[D / 16][4];
  load_q<D>(qa, q + (static_cast<size_t>(b) * q_heads + head0) * D, D, rows);
  float o[D / 8][4];
#pragma unroll
  for (int dn = 0; dn < D / 8; ++dn)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[dn][e] = 0.f;
  for (int p = p_begin; p < p_end; ++p) {
    const int stage = (p - p_begin) & 1;
    cp_async_wait<0>();  // page p is here
    __syncthreads();     // ... for every thread, and everyone is done with page p - 1
    if (p + 1 < p_end) issue(p + 1, stage ^ 1);
    float s[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[nt][e] = 0.f;
    scores<D, 2>(s, qa, Ks + stage * TILE + 16 * warp * STRIDE);
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = p * kTile + 16 * warp + 8 * nt + 2 * t + (e & 1);
        const bool visible = key < len && key >= first_key && g + 8 * (e >> 1) < rows;
        s[nt][e] = visible ? weight_of(fmaf(s[nt][e], negated, add[e >> 1])) : 0.f;
      }
    weighted_values<D, 2>(o, s, Vs + stage * TILE + 16 * warp * STRIDE);
  }
  // The warps' sums meet in shared memory (which the tiles no longer need), the CTAs' sums in
  // distributed shared memory: sums[warp][row][D], then added over warps into sums[0].
  __syncthreads();
  float* sums = reinterpret_cast<float*>(smem_raw);
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    float* dst = sums + (warp * 16 + g + 8 * half) * D;
#pragma unroll
    for (int dn = 0; dn < D / 8; ++dn)
      *reinterpret_cast<float2*>(dst + 8 * dn + 2 * t) = make_float2(o[dn][2 * half], o[dn][2 * half + 1]);
  }
  __syncthreads();
  const int items = rows * D;
  for (int i = threadIdx.x; i < items; i += kThreads) {
    float v = sums[i];
#pragma unroll
    for (int w = 1; w < kThreads / 32; ++w) v += sums[w * 16 * D + i];
    sums[i] = v;  // only this thread reads or writes element i of any warp's part here
  }
  const size_t gate_at = static_cast<size_t>(b) * out.gate_stride + static_cast<size_t>(head0) * D;
  __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(out.out) + static_cast<size_t>(b) * out.stride + head0 * D;
  if (ranks == 1) {
    for (int i = threadIdx.x; i < items; i += kThreads)
      dst[i] = __float2bfloat16_rn(gated(sums[i], out.gate, gate_at + i, out.scale));
    return;
  }
  cg::cluster_group cluster = cg::this_cluster();
  cluster.sync();  // every CTA's sums are complete
  const int share = (items + ranks - 1) / ranks, to = min(items, (rank + 1) * share);
  for (int i = rank * share + threadIdx.x; i < to; i += kThreads) {
    float v = 0.f;
    for (int r = 0; r < ranks; ++r) v += cluster.map_shared_rank(sums, r)[i];
    dst[i] = __float2bfloat16_rn(gated(v, out.gate, gate_at + i, out.scale));
  }
  cluster.sync();  // nobody leaves while a peer may still read its sums
}

template <int D> int tiles_bytes() {
  const int tiles = 4 * kTile * (D + 8) * 2, sums = (kThreads / 32) * 16 * D * 4;
  return tiles > sums ? tiles : sums;
}

template <int D, bool PAGED>
int launch_tiled(const void* q, const void* k, const void* v, const Output& out, const int* cu_seqlens,
                 const int* page_table, int table_stride, const int* slots, const int* kv_lens, int seqs,
                 int max_seq_len, int q_heads, int kv_heads, float scale, int window, const float* offset,
                 cudaStream_t stream) {
  auto kernel = sigmoid_tiled_kernel<D, PAGED>;
  const int bytes = tiles_bytes<D>(), tiles = (max_seq_len + kTile - 1) / kTile;
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return static_cast<int>(e);
  if (seqs > 65535 || tiles > 65535) return LRM_UNSUPPORTED;
  LRM_LAUNCH(kernel, dim3(q_heads, seqs, tiles), kThreads, bytes, stream, static_cast<const __nv_bfloat16*>(q),
             static_cast<const __nv_bfloat16*>(k), static_cast<const __nv_bfloat16*>(v), out, cu_seqlens, page_table,
             table_stride, slots, kv_lens, q_heads, kv_heads, scale, window, offset);
  return 0;
}

template <int D>
int launch_decode(const void* q, const void* k_pages, const void* v_pages, const Output& out, const int* page_table,
                  int table_stride, const int* slots, const int* kv_lens, int seqs, int q_heads, int kv_heads,
                  float scale, int window, const float* offset, int ranks, cudaStream_t stream) {
  auto kernel = sigmoid_decode_kernel<D>;
  const int bytes = tiles_bytes<D>();
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return static_cast<int>(e);
  const int row_groups = (q_heads / kv_heads + 15) / 16;
  const long long clusters = static_cast<long long>(seqs) * kv_heads * row_groups;
  if (clusters > 65535) return LRM_UNSUPPORTED;
  cudaLaunchConfig_t config = {};
  config.gridDim = dim3(ranks, static_cast<unsigned>(clusters));
  config.blockDim = dim3(kThreads);
  config.dynamicSmemBytes = bytes;
  config.stream = stream;
  cudaLaunchAttribute attributes[2];
  attributes[0].id = cudaLaunchAttributeClusterDimension;
  attributes[0].val.clusterDim.x = ranks;
  attributes[0].val.clusterDim.y = 1;
  attributes[0].val.clusterDim.z = 1;
  attributes[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attributes[1].val.programmaticStreamSerializationAllowed = 1;
  config.attrs = attributes;
  config.numAttrs = g_lrm_pdl ? 2 : 1;
  e = cudaLaunchKernelEx(&config, kernel, static_cast<const __nv_bfloat16*>(q),
                         static_cast<const __nv_bfloat16*>(k_pages), static_cast<const __nv_bfloat16*>(v_pages), out,
                         page_table, table_stride, slots, kv_lens, q_heads, kv_heads, row_groups, scale, window, offset);
  return e == cudaSuccess ? 0 : static_cast<int>(e);
}

bool bad_heads(int q_heads, int kv_heads, int d, int dv) {
  return q_heads <= 0 || kv_heads <= 0 || q_heads % kv_heads != 0 || d <= 0 || dv <= 0;
}

}  // namespace

// 1 when the tiled kernels take these head sizes with pages of this many tokens.
LRM_API int lrm_attention_sigmoid_supports(int d, int dv, int page_size) {
  return d == dv && (d == 32 || d == 64 || d == 96 || d == 128) && page_size == kTile ? 1 : 0;
}

// q [T, q_heads, d]. Packed keys (page_table null): k, v [T, kv_heads, d | dv] of the step's own tokens,
// cu_seqlens, seq_of_token [T]. Paged: k, v the cache's pages, slots, and per query seq_of_token and
// positions (int32 [T]) or, with both null, one query per sequence at position kv_lens[b] - 1.
// out [T, out_stride] of `dtype`; gate float32 (pointer at its first column) or null; offset float32 [q_heads].
LRM_API int lrm_attention_sigmoid_rowwise(const void* q, const void* k, const void* v, void* out, int dtype,
                                          long long out_stride, const int* cu_seqlens, const int* seq_of_token,
                                          const int* positions, const int* page_table, int table_stride,
                                          const int* slots, const int* kv_lens, int tokens, int q_heads, int kv_heads,
                                          int d, int dv, int page_size, float scale, int window, const float* offset,
                                          const float* gate, long long gate_stride, float out_scale,
                                          cudaStream_t stream) {
  if (tokens <= 0) return 0;
  const bool paged = page_table != nullptr;
  if (bad_heads(q_heads, kv_heads, d, dv) || offset == nullptr || out_stride < static_cast<long long>(q_heads) * dv)
    return LRM_BAD_ARGUMENT;
  if (paged ? (slots == nullptr || page_size <= 0 || (seq_of_token == nullptr) != (positions == nullptr) ||
               (positions == nullptr && kv_lens == nullptr))
            : (cu_seqlens == nullptr || seq_of_token == nullptr))
    return LRM_BAD_ARGUMENT;
  if (q_heads > 65535 || d > 1024 || dv > 1024) return LRM_UNSUPPORTED;
  const dim3 grid(tokens, q_heads);
  const int widest = d > dv ? d : dv;
  const Output o{out, out_stride, gate, gate_stride, out_scale};
#define LRM_ROWS(AT, PER, PG)                                                                                   \
  LRM_LAUNCH((sigmoid_rowwise_kernel<AT, PER, PG>), grid, 32, 0, stream, static_cast<const AT*>(q),             \
             static_cast<const AT*>(k), static_cast<const AT*>(v), o, cu_seqlens, seq_of_token, positions,      \
             page_table, table_stride, slots, kv_lens, q_heads, kv_heads, d, dv, page_size, scale, window, offset)
#define LRM_ROWS_BY_WIDTH(AT)                                                        \
  do {                                                                               \
    if (widest <= 128) { if (paged) LRM_ROWS(AT, 4, true); else LRM_ROWS(AT, 4, false); }  \
    else if (widest <= 256) { if (paged) LRM_ROWS(AT, 8, true); else LRM_ROWS(AT, 8, false); }  \
    else { if (paged) LRM_ROWS(AT, 32, true); else LRM_ROWS(AT, 32, false); }        \
  } while (0)
  if (dtype == LRM_F32)
    LRM_ROWS_BY_WIDTH(float);
  else if (dtype == LRM_BF16)
    LRM_ROWS_BY_WIDTH(__nv_bfloat16);
  else
    return LRM_BAD_ARGUMENT;
#undef LRM_ROWS_BY_WIDTH
#undef LRM_ROWS
  return 0;
}

#define LRM_BY_HEAD_SIZE(CALL) \
  switch (d) {                 \
    case 32: return CALL(32);  \
    case 64: return CALL(64);  \
    case 96: return CALL(96);  \
    case 128: return CALL(128); \
    default: return LRM_UNSUPPORTED; \
  }

// bfloat16; sequences' queries are rows cu_seqlens[b] .. cu_seqlens[b + 1] - 1 of q [T, q_heads, d], at most
// max_seq_len of them. With a page table the keys (kv_lens[b] of them, the step's own included) are in the
// cache, without one k and v are the step's packed own.
LRM_API int lrm_attention_sigmoid_tiled(const void* q, const void* k, const void* v, void* out, long long out_stride,
                                        const int* cu_seqlens, const int* page_table, int table_stride,
                                        const int* slots, const int* kv_lens, int seqs, int max_seq_len, int q_heads,
                                        int kv_heads, int d, float scale, int window, const float* offset,
                                        const float* gate, long long gate_stride, float out_scale,
                                        cudaStream_t stream) {
  if (seqs <= 0 || max_seq_len <= 0) return 0;
  if (bad_heads(q_heads, kv_heads, d, d) || offset == nullptr || cu_seqlens == nullptr ||
      (page_table != nullptr && (slots == nullptr || kv_lens == nullptr)))
    return LRM_BAD_ARGUMENT;
  if (out_stride % 2 != 0 || reinterpret_cast<uintptr_t>(out) % 4 != 0) return LRM_UNSUPPORTED;
  const Output o{out, out_stride, gate, gate_stride, out_scale};
#define LRM_TILED(DIM)                                                                                               \
  (page_table != nullptr                                                                                             \
       ? launch_tiled<DIM, true>(q, k, v, o, cu_seqlens, page_table, table_stride, slots, kv_lens, seqs, max_seq_len, \
                                 q_heads, kv_heads, scale, window, offset, stream)                                   \
       : launch_tiled<DIM, false>(q, k, v, o, cu_seqlens, nullptr, 0, nullptr, nullptr, seqs, max_seq_len, q_heads,  \
                                  kv_heads, scale, window, offset, stream))
  LRM_BY_HEAD_SIZE(LRM_TILED)
#undef LRM_TILED
}

// bfloat16, one query per sequence (q [seqs, q_heads, d]) over the cache; `ranks` (1 to 8): CTAs that share
// a sequence's keys.
LRM_API int lrm_attention_sigmoid_decode(const void* q, const void* k_pages, const void* v_pages, void* out,
                                         long long out_stride, const int* page_table, int table_stride,
                                         const int* slots, const int* kv_lens, int seqs, int q_heads, int kv_heads,
                                         int d, float scale, int window, const float* offset, const float* gate,
                                         long long gate_stride, float out_scale, int ranks, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (bad_heads(q_heads, kv_heads, d, d) || offset == nullptr || page_table == nullptr || slots == nullptr ||
      kv_lens == nullptr || ranks < 1 || ranks > 8)
    return LRM_BAD_ARGUMENT;
  const Output o{out, out_stride, gate, gate_stride, out_scale};
#define LRM_DECODE(DIM)                                                                                             \
  launch_decode<DIM>(q, k_pages, v_pages, o, page_table, table_stride, slots, kv_lens, seqs, q_heads, kv_heads, scale, \
                     window, offset, ranks, stream)
  LRM_BY_HEAD_SIZE(LRM_DECODE)
#undef LRM_DECODE
}
