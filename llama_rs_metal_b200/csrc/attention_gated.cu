// Causal grouped-query softmax attention for layers that go beyond the plain form, each step only if asked for:
//   s = scale * (q . k);  s <- cap * tanh(s / cap)                        a cap on the scores
//   key j is visible to the query at p:  j <= p and (j >= first_visible_key(p, window) or j < keep)
//                                         a window (or a chunk of positions), and kept first keys besides
//   w = softmax over the visible keys, whose denominator also holds exp(sink_h)
//   out = (sum_j w_j v_j) * sigmoid(gate) * out_scale                     a gate per head and value dimension,
//                                                                         or one number per head
// Scores, weights, sums and the gate (pre-activations in float32, read where the result leaves the kernel) are
// float32. Keys and values have widths of their own (d, dv). The result of token t, head h goes to
// out[t * out_stride + h * dv]: a column range of a wider row, so that a product can read it beside others.
//
//  * row-wise: one warp per (query, head), keys one at a time in ascending order, from the step's packed
//    keys or the paged cache, both dtypes, head sizes up to 1024: the attention of the float32 path, and
//    of sizes the tiled kernels refuse.
//  * tiled (bfloat16, d and dv multiples of 8 up to 128, filled up with zeros to 32, 64, 96 or 128 in shared
//    memory): 64 queries of one head per CTA over 64-key tiles on mma.sync, double buffered by cp.async, from
//    packed keys (prompts) or the cache's pages (portions). The tiles of the kept keys come first, then those
//    of the window; tiles that every query sees whole take no test per score. (Prompts mostly run
//    attention_gated_umma.cu.)
//  * decode (same sizes): one query per sequence over the cache; the CTAs of a thread-block cluster take runs
//    of the visible pages, and their sums, maxima and masses meet in distributed shared memory in rank order:
//    one launch, no partial rows in memory. It can begin at the float32 projection (Fresh): it then adds the
//    biases, rotates the queries and the new key, and stores the new key and value in the cache itself, with
//    the arithmetic of shaped_qkv.cu.
// Rows of a tile that nobody sees are zero-filled on the way into shared memory, so stale cache contents never
// reach a product.
#include <cooperative_groups.h>

#include "attention_gated.cuh"
#include "attention_mma.cuh"

namespace {

namespace cg = cooperative_groups;

constexpr int kStages = 3;    // pages of a decode step's ring
constexpr int kMaxRanks = 8;  // CTAs that share a sequence's keys in a decode step, at most

static_assert(kTile == kKeyTile, "a tile of keys is a page");

// Where keys come from: packed rows of the step (table null) or the cache's pages.
struct Source {
  const void* k;
  const void* v;
  const int* page_table;
  int table_stride;
  const int* slots;
  const int* kv_lens;
};

// The step's projection rows [q_heads * d | kv_heads * d | kv_heads * dv | ...], for a decode step that splits them
// in the attention kernel. Rotation: dimension i of the first `rotary` of a head with i + rotary / 2.
struct Fresh {
  const float* proj;        // row b at proj + b * stride; null: q, k and v were split before
  long long stride;
  const float* bias;        // [row] or null
  const float2* table;      // [seqs, rotary / 2] (cos, sin), or null
  int rotary;
  const int* dest_rows;     // [seqs]: page * 64 + row of the new token in the cache
};

// --------------------------------------------------------------------------- row-wise
template <typename A, int PER, bool PAGED>
__global__ void gated_rowwise_kernel(const A* q, Source src, Form f, const int* __restrict__ cu_seqlens,
                                     const int* __restrict__ seq_of_token, const int* __restrict__ positions,
                                     int q_heads, int kv_heads, int d, int dv, int page_size) {
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, kh = h / (q_heads / kv_heads);
  const int lane = threadIdx.x & 31;
  int pos, start = 0;
  const int* table = nullptr;
  if (PAGED) {
    const int b = seq_of_token != nullptr ? seq_of_token[t] : t;
    pos = positions != nullptr ? positions[t] : src.kv_lens[b] - 1;
    table = src.page_table + static_cast<size_t>(src.slots[b]) * src.table_stride;
  } else {
    start = cu_seqlens[seq_of_token[t]];
    pos = t - start;
  }
  const A* qr = q + (static_cast<size_t>(t) * q_heads + h) * d;
  float qv[PER], acc[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int j = lane + 32 * i;
    qv[i] = j < d ? to_f32(qr[j]) : 0.f;
    acc[i] = 0.f;
  }
  // a sink is a key met before all others: score `sink`, weight 1 at its own maximum, no value
  float m = f.sinks != nullptr ? f.sinks[h] : -INFINITY, l = f.sinks != nullptr ? 1.f : 0.f;
  const int first = first_visible_key(pos, f.window), kept = min(f.keep, first);
  for (int i = 0, n = kept + pos - first + 1; i < n; ++i) {
    const int p = i < kept ? i : first + i - kept;
    size_t key;  // row number among rows of one key head's width
    if (PAGED) {
      const int page = table[p / page_size];
      key = (static_cast<size_t>(page) * kv_heads + kh) * page_size + p % page_size;
    } else {
      key = static_cast<size_t>(start + p) * kv_heads + kh;
    }
    const A* kr = static_cast<const A*>(src.k) + key * d;
    const A* vr = static_cast<const A*>(src.v) + key * dv;
    float dot = 0.f;
#pragma unroll
    for (int e = 0; e < PER; ++e) {
      const int j = lane + 32 * e;
      if (j < d) dot = fmaf(qv[e], to_f32(kr[j]), dot);
    }
    float s = warp_sum(dot) * f.scale;
    if (f.cap > 0.f) s = f.cap * tanhf(s / f.cap);
    const float nm = fmaxf(m, s);
    const float old = expf(m - nm), prob = expf(s - nm);
    l = fmaf(l, old, prob);
#pragma unroll
    for (int e = 0; e < PER; ++e) {
      const int j = lane + 32 * e;
      if (j < dv) acc[e] = fmaf(prob, to_f32(vr[j]), __fmul_rn(acc[e], old));
    }
    m = nm;
  }
  A* dst = static_cast<A*>(f.out) + static_cast<size_t>(t) * f.out_stride + h * dv;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int j = lane + 32 * i;
    if (j < dv) dst[j] = from_f32<A>(acc[i] / l * gate_at(f, t, h, dv, j));
  }
}

// --------------------------------------------------------------------------- tiles
template <int N>
__device__ __forceinline__ void to_scores(float (&s)[N][4], const ScoreMap& map) {
  if (map.capped) {
#pragma unroll
    for (int nt = 0; nt < N; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[nt][e] = map.cap(s[nt][e]);
  } else {
#pragma unroll
    for (int nt = 0; nt < N; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[nt][e] = map.plain(s[nt][e]);
  }
}

// Rows [lo, hi) of 64 x width elements (row pitch `pitch`) into a padded tile of D columns; everything else of
// the tile is zero-filled.
template <int D>
__device__ __forceinline__ void load_rows(__nv_bfloat16* dst, const __nv_bfloat16* src, size_t pitch, int width, int lo, int hi) {
  constexpr int STRIDE = D + 8, CHUNKS = D / 8;
#pragma unroll 4
  for (int idx = threadIdx.x; idx < kTile * CHUNKS; idx += kThreads) {
    const int r = idx / CHUNKS, c = (idx % CHUNKS) * 8;
    const bool ok = r >= lo && r < hi && c < width;
    cp_async16(dst + r * STRIDE + c, ok ? src + r * pitch + c : src, ok ? 16 : 0);
  }
}

// Query fragments of 16 rows x D, of which `width` columns exist: row r lives at base + r * pitch.
template <int D>
__device__ __forceinline__ void load_queries(uint32_t (&qa)[D / 16][4], const __nv_bfloat16* base, size_t pitch, int width,
                                             int valid_rows) {
  const int lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int ks = 0; ks < D / 16; ++ks)
#pragma unroll
    for (int half = 0; half < 2; ++half)
#pragma unroll
      for (int hi = 0; hi < 2; ++hi) {
        const int r = g + 8 * half, c = 16 * ks + 8 * hi + 2 * t;
        qa[ks][half + 2 * hi] = r < valid_rows && c < width ? *reinterpret_cast<const uint32_t*>(base + r * pitch + c) : 0u;
      }
}

template <int D, int DV>
__global__ __launch_bounds__(kThreads) void gated_tiled_kernel(const __nv_bfloat16* q, Source src, Form f,
                                                               const int* __restrict__ cu_seqlens, int q_heads,
                                                               int kv_heads, int d, int dv) {
  constexpr int KTILE = kTile * (D + 8), VTILE = kTile * (DV + 8);
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(smem_raw);  // [2][64][D + 8]
  __nv_bfloat16* Vs = Ks + 2 * KTILE;                              // [2][64][DV + 8]

  const bool paged = src.page_table != nullptr;
  const int qt = gridDim.z - 1 - blockIdx.z;  // the longest rows of work first
  const int h = blockIdx.x, b = blockIdx.y;
  const int start = cu_seqlens[b], n = cu_seqlens[b + 1] - start;
  const int q0 = qt * kTile;
  if (q0 >= n) return;
  const int len = paged ? src.kv_lens[b] : n, before = len - n;
  const int kh = h / (q_heads / kv_heads);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int row0 = q0 + 16 * warp;  // this warp's first query, counted within the portion
  const int* table = paged ? src.page_table + static_cast<size_t>(src.slots[b]) * src.table_stride : nullptr;
  const ScoreMap map(f);
  const float sink_log2 = f.sinks != nullptr ? f.sinks[h] * kLog2e : -INFINITY;
  pdl_wait();

  uint32_t qa[D / 16][4];
  load_queries<D>(qa, q + (static_cast<size_t>(start + row0) * q_heads + h) * d, static_cast<size_t>(q_heads) * d, d, n - row0);
  float o[DV / 8][4];
#pragma unroll
  for (int dn = 0; dn < DV / 8; ++dn)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[dn][e] = 0.f;
  // a sink: the row's softmax starts from the maximum sink and the mass 1 (held by one lane of four)
  const float l0 = (f.sinks != nullptr && t == 0) ? 1.f : 0.f;
  float m[2] = {sink_log2, sink_log2}, l[2] = {l0, l0};

  const int last = before + min(q0 + kTile, n) - 1;  // the CTA's last query
  const int first_key = first_visible_key(before + q0, f.window);
  const Tiles tiles(first_key, last, f.keep);
  const int query[2] = {before + row0 + g, before + row0 + g + 8};
  const int row_first[2] = {first_visible_key(query[0], f.window), first_visible_key(query[1], f.window)};
  // tiles all of whose keys every query of the CTA sees need no test per score
  const int whole_from = first_visible_key(last, f.window), whole_to = before + q0;
  const size_t k_pitch = paged ? d : static_cast<size_t>(kv_heads) * d, v_pitch = paged ? dv : static_cast<size_t>(kv_heads) * dv;
  auto issue = [&](int i, int stage) {
    const int kt = tiles.at(i), k0 = kt * kTile;
    const int lo = k0 < f.keep ? 0 : first_key - k0;
    int hi = i < tiles.kept ? f.keep - k0 : len - k0;
    size_t row;  // of the tile's first key, among rows of one key head
    if (paged) {
      const int page = table[kt];
      if (page < 0) hi = 0;
      row = (static_cast<size_t>(max(page, 0)) * kv_heads + kh) * kTile;
    } else {
      row = static_cast<size_t>(start + k0) * kv_heads + kh;
    }
    load_rows<D>(Ks + stage * KTILE, static_cast<const __nv_bfloat16*>(src.k) + row * d, k_pitch, d, lo, hi);
    load_rows<DV>(Vs + stage * VTILE, static_cast<const __nv_bfloat16*>(src.v) + row * dv, v_pitch, dv, lo, hi);
    cp_async_commit();
  };
  issue(0, 0);
  for (int i = 0; i < tiles.count; ++i) {
    const int stage = i & 1, k0 = tiles.at(i) * kTile;
    if (i + 1 < tiles.count) {
      issue(i + 1, stage ^ 1);
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
    scores<D, 8>(s, qa, Ks + stage * KTILE);
    to_scores(s, map);
    if (k0 + kTile - 1 > whole_to || (k0 < whole_from && k0 + kTile > f.keep)) {
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (!sees(f, k0 + 8 * nt + 2 * t + (e & 1), query[e >> 1], row_first[e >> 1])) s[nt][e] = -INFINITY;
    }
    softmax_update<DV, 8>(s, o, m, l);
    weighted_values<DV, 8>(o, s, Vs + stage * VTILE);
    __syncthreads();
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    float total = l[half];
    total += __shfl_xor_sync(0xffffffffu, total, 1);
    total += __shfl_xor_sync(0xffffffffu, total, 2);
    const int row = row0 + g + 8 * half;
    if (row >= n) continue;
    const size_t tok = static_cast<size_t>(start + row);
    const float inv = 1.0f / total;
    __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(f.out) + tok * f.out_stride + h * dv;
    const bool by_element = f.gate != nullptr && !f.gate_per_head;
    const float head_gate = by_element ? inv : inv * gate_at(f, tok, h, dv, 0);
#pragma unroll
    for (int dn = 0; dn < DV / 8; ++dn) {
      const int c = 8 * dn + 2 * t;
      if (c >= dv) continue;
      float a = head_gate, e = head_gate;
      if (by_element) {
        const float* z = f.gate + tok * f.gate_stride + h * dv + c;
        a *= f.out_scale * unit_sigmoid(z[0]);
        e *= f.out_scale * unit_sigmoid(z[1]);
      }
      *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(o[dn][2 * half] * a, o[dn][2 * half + 1] * e);
    }
  }
}

// --------------------------------------------------------------------------- decode
// A cluster of gridDim.x CTAs per (sequence, kv head, group of up to 16 query heads) [blockIdx.y]; the
// CTA of rank r takes a run of the visible pages, its four warps 16 keys of every page each.
template <int D, int DV>
__global__ __launch_bounds__(kThreads) void gated_decode_kernel(const __nv_bfloat16* q, Source src, Form f, Fresh fresh,
                                                                int q_heads, int kv_heads, int row_groups, int d, int dv) {
  constexpr int KSTRIDE = D + 8, VSTRIDE = DV + 8, KTILE = kTile * KSTRIDE, VTILE = kTile * VSTRIDE;
  constexpr int PART = DV + 2;  // a row's sums, maximum (log2 domain) and mass
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(smem_raw);  // [kStages][64][D + 8]
  __nv_bfloat16* Vs = Ks + kStages * KTILE;                        // [kStages][64][DV + 8]
  const int ranks = gridDim.x, rank = blockIdx.x;
  const int rg = blockIdx.y % row_groups, kh = (blockIdx.y / row_groups) % kv_heads;
  const int b = blockIdx.y / (row_groups * kv_heads);
  const int group = q_heads / kv_heads, head0 = kh * group + 16 * rg;
  const int rows = min(16, group - 16 * rg);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int len = src.kv_lens[b], query = len - 1;
  const int first_key = first_visible_key(max(query, 0), f.window);
  const Tiles tiles(first_key, max(query, 0), f.keep);
  const int count = len > 0 ? tiles.count : 0;
  const int per_rank = (count + ranks - 1) / ranks;
  const int begin = min(count, rank * per_rank), end = min(count, begin + per_rank);
  const int* table = src.page_table + static_cast<size_t>(src.slots[b]) * src.table_stride;
  const ScoreMap map(f);

  auto issue = [&](int i) {  // page i of the list into its stage; one group of copies per call, empty beyond the end
    if (i >= end) {
      cp_async_commit();
      return;
    }
    const int stage = (i - begin) % kStages;
    const int page_index = tiles.at(i), k0 = page_index * kTile, page = table[page_index];
    const int lo = k0 < f.keep ? 0 : first_key - k0;
    const int hi = page < 0 ? 0 : i < tiles.kept ? f.keep - k0 : len - k0;
    const size_t row = (static_cast<size_t>(max(page, 0)) * kv_heads + kh) * kTile;
    load_rows<D>(Ks + stage * KTILE, static_cast<const __nv_bfloat16*>(src.k) + row * d, d, d, lo, hi);
    load_rows<DV>(Vs + stage * VTILE, static_cast<const __nv_bfloat16*>(src.v) + row * dv, dv, dv, lo, hi);
    cp_async_commit();
  };
  // only q and the newest key and value row (in the last page) come from the kernel before this one; where
  // this kernel splits the projection it puts the newest row there itself
  const bool split = fresh.proj != nullptr;
  int issued = begin;
  while (issued < begin + kStages - 1 && (split || issued < count - 1)) issue(issued++);
  pdl_wait();
  while (issued < begin + kStages - 1) issue(issued++);

  uint32_t qa[D / 16][4];
  __nv_bfloat16* Qs = Vs + kStages * VTILE;  // [16][D + 8], behind it the new key [D] and the new value [DV]
  __nv_bfloat16* new_key = Qs + 16 * KSTRIDE;
  __nv_bfloat16* new_value = new_key + D;
  const bool has_newest = split && end == count && begin < end;
  if (split) {
    // columns of this CTA's query heads, then of the new key and of the new value, kItems at a time so that their
    // loads are all under way before the first is used
    constexpr int kItems = 4;
    const float* row = fresh.proj + static_cast<size_t>(b) * fresh.stride;
    const int half = fresh.rotary / 2;
    const float2* turns = fresh.table + static_cast<size_t>(b) * half;
    const int nq = rows * d, items = nq + (has_newest ? d + dv : 0);
    const int dest = has_newest && rg == 0 ? fresh.dest_rows[b] : -1;  // one of the groups of query heads stores the row
    const size_t cached = dest >= 0 ? (static_cast<size_t>(dest / kTile) * kv_heads + kh) * kTile + dest % kTile : 0;
    __nv_bfloat16* k_row = const_cast<__nv_bfloat16*>(static_cast<const __nv_bfloat16*>(src.k)) + cached * d;
    __nv_bfloat16* v_row = const_cast<__nv_bfloat16*>(static_cast<const __nv_bfloat16*>(src.v)) + cached * dv;
    for (int i0 = threadIdx.x; i0 < items; i0 += kItems * kThreads) {
      float x[kItems], partner[kItems];
      float2 turn[kItems];
      int place[kItems];  // column within its head
#pragma unroll
      for (int u = 0; u < kItems; ++u) {
        const int i = i0 + u * kThreads;
        const bool is_v = i >= nq + d;
        const int col = i < nq ? head0 * d + i : is_v ? (q_heads + kv_heads) * d + kh * dv + i - nq - d : (q_heads + kh) * d + i - nq;
        const int c = i < nq ? i % d : is_v ? i - nq - d : i - nq;
        place[u] = c;
        x[u] = partner[u] = 0.f;
        turn[u] = make_float2(1.f, 0.f);
        if (i >= items) continue;
        x[u] = row[col] + (fresh.bias != nullptr ? fresh.bias[col] : 0.f);
        if (!is_v && c < 2 * half) {
          const int other = c < half ? col + half : col - half;
          partner[u] = row[other] + (fresh.bias != nullptr ? fresh.bias[other] : 0.f);
          turn[u] = turns[c < half ? c : c - half];
        }
      }
#pragma unroll
      for (int u = 0; u < kItems; ++u) {
        const int i = i0 + u * kThreads, c = place[u];
        if (i >= items) continue;
        const float cross = __fmul_rn(partner[u], turn[u].y);
        const __nv_bfloat16 y = __float2bfloat16_rn(i >= nq + d || c >= 2 * half ? x[u] : fmaf(x[u], turn[u].x, c < half ? -cross : cross));
        if (i < nq) {
          Qs[(i / d) * KSTRIDE + c] = y;
        } else if (i < nq + d) {
          new_key[c] = y;
          if (dest >= 0) k_row[c] = y;
        } else {
          new_value[c] = y;
          if (dest >= 0) v_row[c] = y;
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = g + 8 * (e & 1), c = 16 * ks + 8 * (e >> 1) + 2 * t;
        qa[ks][e] = r < rows && c < d ? *reinterpret_cast<const uint32_t*>(Qs + r * KSTRIDE + c) : 0u;
      }
  } else {
    load_queries<D>(qa, q + (static_cast<size_t>(b) * q_heads + head0) * d, d, d, rows);
  }
  float o[DV / 8][4];
#pragma unroll
  for (int dn = 0; dn < DV / 8; ++dn)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[dn][e] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  for (int i = begin; i < end; ++i) {
    const int stage = (i - begin) % kStages, k0 = tiles.at(i) * kTile + 16 * warp;
    cp_async_wait<kStages - 2>();  // page i is here
    __syncthreads();               // ... for every thread, and everyone is done with page i - 1
    issue(i + kStages - 1);
    if (has_newest && i == count - 1) {  // the page's copy of the newest row is older than the row
      const int r = query % kTile;
      for (int c = threadIdx.x; c < d + dv; c += kThreads) {
        if (c < d) Ks[stage * KTILE + r * KSTRIDE + c] = new_key[c];
        else Vs[stage * VTILE + r * VSTRIDE + c - d] = new_value[c - d];
      }
      __syncthreads();
    }
    float s[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[nt][e] = 0.f;
    scores<D, 2>(s, qa, Ks + stage * KTILE + 16 * warp * KSTRIDE);
    to_scores(s, map);
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (!sees(f, k0 + 8 * nt + 2 * t + (e & 1), query, first_key)) s[nt][e] = -INFINITY;
    if (rows > 8) softmax_update<DV, 2, 2>(s, o, m, l);
    else softmax_update<DV, 2, 1>(s, o, m, l);  // query heads 8..15 of the tile are padding
    weighted_values<DV, 2>(o, s, Vs + stage * VTILE + 16 * warp * VSTRIDE);
  }
  // The warps' parts meet in shared memory (which the tiles no longer need), the CTAs' parts in distributed
  // shared memory: parts[warp][row][PART], put together into joined[row][PART].
  __syncthreads();
  float* parts = reinterpret_cast<float*>(smem_raw);
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    float total = l[half];
    total += __shfl_xor_sync(0xffffffffu, total, 1);
    total += __shfl_xor_sync(0xffffffffu, total, 2);
    float* dst = parts + (warp * 16 + g + 8 * half) * PART;
#pragma unroll
    for (int dn = 0; dn < DV / 8; ++dn)
      *reinterpret_cast<float2*>(dst + 8 * dn + 2 * t) = make_float2(o[dn][2 * half], o[dn][2 * half + 1]);
    if (t == 0) {
      dst[DV] = m[half];
      dst[DV + 1] = total;
    }
  }
  __syncthreads();
  float* joined = parts + (kThreads / 32) * 16 * PART;
  for (int i = threadIdx.x; i < rows * PART; i += kThreads) {
    const int r = i / PART, c = i % PART;
    float top = -INFINITY, value = 0.f;
#pragma unroll
    for (int w = 0; w < kThreads / 32; ++w) top = fmaxf(top, parts[(w * 16 + r) * PART + DV]);
#pragma unroll
    for (int w = 0; w < kThreads / 32; ++w) {
      const float mw = parts[(w * 16 + r) * PART + DV];
      if (mw > -INFINITY) value = fmaf(parts[(w * 16 + r) * PART + c], exp2_fast(mw - top), value);
    }
    joined[i] = c == DV ? top : value;
  }
  cg::cluster_group cluster = cg::this_cluster();
  const int outputs = rows * dv, share = (outputs + ranks - 1) / ranks, to = min(outputs, (rank + 1) * share);
  const int mine = rank * share + threadIdx.x;  // the first of this thread's outputs: its gate comes while the others arrive
  float gate = mine < to ? gate_at(f, b, head0 + mine / dv, dv, mine % dv) : 0.f;
  if (ranks > 1) cluster.sync();  // every CTA's parts are complete
  else __syncthreads();
  __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(f.out) + static_cast<size_t>(b) * f.out_stride + head0 * dv;
  for (int i = mine; i < to; i += kThreads) {
    const int r = i / dv, c = i % dv;
    if (i != mine) gate = gate_at(f, b, head0 + r, dv, c);
    const float sink_log2 = f.sinks != nullptr ? f.sinks[head0 + r] * kLog2e : -INFINITY;
    float mk[kMaxRanks], lk[kMaxRanks], vk[kMaxRanks];  // all of the peers' values under way together
#pragma unroll
    for (int k = 0; k < kMaxRanks; ++k) {
      const float* part = cluster.map_shared_rank(joined, k < ranks ? k : 0) + r * PART;
      mk[k] = k < ranks ? part[DV] : -INFINITY;
      lk[k] = k < ranks ? part[DV + 1] : 0.f;
      vk[k] = k < ranks ? part[c] : 0.f;
    }
    float top = sink_log2, value = 0.f;
#pragma unroll
    for (int k = 0; k < kMaxRanks; ++k) top = fmaxf(top, mk[k]);
    float mass = f.sinks != nullptr ? exp2f(sink_log2 - top) : 0.f;
#pragma unroll
    for (int k = 0; k < kMaxRanks; ++k)
      if (mk[k] > -INFINITY) {  // (a CTA that saw no key has nothing to add)
        const float w = exp2f(mk[k] - top);
        value = fmaf(vk[k], w, value);
        mass = fmaf(lk[k], w, mass);
      }
    dst[i] = __float2bfloat16_rn(value / mass * gate);
  }
  if (ranks > 1) cluster.sync();  // nobody leaves while a peer may still read its parts
}

template <int D, int DV> constexpr int tiles_bytes() { return 2 * kTile * (D + 8 + DV + 8) * 2; }
template <int D, int DV> constexpr int fresh_bytes() { return (16 * (D + 8) + D + DV) * 2; }
template <int DV> constexpr int parts_bytes() { return (kThreads / 32 + 1) * 16 * (DV + 2) * 4; }

struct Geometry {
  int seqs, max_seq_len, q_heads, kv_heads, d, dv, ranks;
  Fresh fresh;
};

template <int D, int DV>
int launch_tiled(const void* q, const Source& src, const Form& f, const int* cu_seqlens, const Geometry& g, cudaStream_t stream) {
  auto kernel = gated_tiled_kernel<D, DV>;
  const int bytes = tiles_bytes<D, DV>(), tiles = (g.max_seq_len + kTile - 1) / kTile;
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return static_cast<int>(e);
  if (g.seqs > 65535 || tiles > 65535) return LRM_UNSUPPORTED;
  LRM_LAUNCH(kernel, dim3(g.q_heads, g.seqs, tiles), kThreads, bytes, stream, static_cast<const __nv_bfloat16*>(q), src, f,
             cu_seqlens, g.q_heads, g.kv_heads, g.d, g.dv);
  return 0;
}

template <int D, int DV>
int launch_decode(const void* q, const Source& src, const Form& f, const int*, const Geometry& g, cudaStream_t stream) {
  auto kernel = gated_decode_kernel<D, DV>;
  const int held = tiles_bytes<D, DV>() / 2 * kStages + (g.fresh.proj != nullptr ? fresh_bytes<D, DV>() : 0);
  const int bytes = held > parts_bytes<DV>() ? held : parts_bytes<DV>();
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return static_cast<int>(e);
  const int row_groups = (g.q_heads / g.kv_heads + 15) / 16;
  const long long clusters = static_cast<long long>(g.seqs) * g.kv_heads * row_groups;
  if (clusters > 65535) return LRM_UNSUPPORTED;
  cudaLaunchConfig_t config = {};
  config.gridDim = dim3(g.ranks, static_cast<unsigned>(clusters));
  config.blockDim = dim3(kThreads);
  config.dynamicSmemBytes = bytes;
  config.stream = stream;
  cudaLaunchAttribute attributes[2];
  attributes[0].id = cudaLaunchAttributeClusterDimension;
  attributes[0].val.clusterDim.x = g.ranks;
  attributes[0].val.clusterDim.y = 1;
  attributes[0].val.clusterDim.z = 1;
  attributes[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attributes[1].val.programmaticStreamSerializationAllowed = 1;
  config.attrs = attributes;
  // a cluster of several CTAs does not start ahead of its predecessor's end: let in early, its CTAs take the places
  // that come free one by one and hold them while the others still wait for theirs (2 to 20 us per decode step)
  config.numAttrs = g_lrm_pdl && g.ranks == 1 ? 2 : 1;
  e = cudaLaunchKernelEx(&config, kernel, static_cast<const __nv_bfloat16*>(q), src, f, g.fresh, g.q_heads, g.kv_heads,
                         row_groups, g.d, g.dv);
  return e == cudaSuccess ? 0 : static_cast<int>(e);
}

}  // namespace

// 1 when the tiled kernels take these head sizes with pages of this many tokens.
LRM_API int lrm_attention_gated_supports(int d, int dv, int page_size) {
  return d > 0 && dv > 0 && d <= 128 && dv <= 128 && d % 8 == 0 && dv % 8 == 0 && page_size == kTile ? 1 : 0;
}

// q [T, q_heads, d]. Packed keys (page_table null): k, v [T, kv_heads, d | dv] of the step's own tokens,
// cu_seqlens, seq_of_token [T]. Paged: k, v the cache's pages, slots, and per query seq_of_token and
// positions (int32 [T]) or, with both null, one query per sequence at position kv_lens[b] - 1.
// out [T, out_stride] of `dtype` (pointer at its first column); gate float32 (likewise) or null.
LRM_API int lrm_attention_gated_rowwise(const void* q, const void* k, const void* v, int dtype, const int* cu_seqlens,
                                        const int* seq_of_token, const int* positions, const int* page_table,
                                        int table_stride, const int* slots, const int* kv_lens, int tokens, int q_heads,
                                        int kv_heads, int d, int dv, int page_size, float scale, float cap, int window,
                                        int keep, const float* sinks, const float* gate, long long gate_stride,
                                        int gate_per_head, void* out, long long out_stride, float out_scale,
                                        cudaStream_t stream) {
  if (tokens <= 0) return 0;
  const bool paged = page_table != nullptr;
  const Form f = make_form(scale, cap, window, keep, sinks, gate, gate_stride, gate_per_head, out, out_stride, out_scale);
  if (bad_form(f, q_heads, kv_heads, d, dv)) return LRM_BAD_ARGUMENT;
  if (paged ? (slots == nullptr || page_size <= 0 || (seq_of_token == nullptr) != (positions == nullptr) ||
               (positions == nullptr && kv_lens == nullptr))
            : (cu_seqlens == nullptr || seq_of_token == nullptr))
    return LRM_BAD_ARGUMENT;
  if (q_heads > 65535 || d > 1024 || dv > 1024) return LRM_UNSUPPORTED;
  const dim3 grid(tokens, q_heads);
  const int widest = d > dv ? d : dv;
  const Source src{k, v, page_table, table_stride, slots, kv_lens};
#define LRM_ROWS(AT, PER, PG)                                                                                            \
  LRM_LAUNCH((gated_rowwise_kernel<AT, PER, PG>), grid, 32, 0, stream, static_cast<const AT*>(q), src, f, cu_seqlens,    \
             seq_of_token, positions, q_heads, kv_heads, d, dv, page_size)
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

#define LRM_BY_VALUE_SIZE(LAUNCH, DIM)                                                          \
  do {                                                                                          \
    if (dv <= 32) return LAUNCH<DIM, 32>(q, src, f, cu_seqlens, g, stream);                     \
    if (dv <= 64) return LAUNCH<DIM, 64>(q, src, f, cu_seqlens, g, stream);                     \
    if (dv <= 96) return LAUNCH<DIM, 96>(q, src, f, cu_seqlens, g, stream);                     \
    return LAUNCH<DIM, 128>(q, src, f, cu_seqlens, g, stream);                                  \
  } while (0)
#define LRM_BY_SIZES(LAUNCH)                          \
  do {                                                \
    if (d <= 32) LRM_BY_VALUE_SIZE(LAUNCH, 32);       \
    if (d <= 64) LRM_BY_VALUE_SIZE(LAUNCH, 64);       \
    if (d <= 96) LRM_BY_VALUE_SIZE(LAUNCH, 96);       \
    LRM_BY_VALUE_SIZE(LAUNCH, 128);                   \
  } while (0)

// bfloat16; sequences' queries are rows cu_seqlens[b] .. cu_seqlens[b + 1] - 1 of q [T, q_heads, d], at most
// max_seq_len of them. With a page table the keys (kv_lens[b] of them, the step's own included) are in the
// cache, without one k and v are the step's packed own. `ranks` > 0 (1 to 8): instead one query per sequence
// (q [seqs, q_heads, d]) over the cache, the keys shared by a cluster of that many CTAs; cu_seqlens is not read.
LRM_API int lrm_attention_gated(const void* q, const void* k, const void* v, const int* cu_seqlens, const int* page_table,
                                int table_stride, const int* slots, const int* kv_lens, int seqs, int max_seq_len, int q_heads,
                                int kv_heads, int d, int dv, float scale, float cap, int window, int keep, const float* sinks,
                                const float* gate, long long gate_stride, int gate_per_head, void* out, long long out_stride,
                                float out_scale, int ranks, cudaStream_t stream) {
  if (seqs <= 0 || (ranks == 0 && max_seq_len <= 0)) return 0;
  const Form f = make_form(scale, cap, window, keep, sinks, gate, gate_stride, gate_per_head, out, out_stride, out_scale);
  if (bad_form(f, q_heads, kv_heads, d, dv) || ranks < 0 || ranks > kMaxRanks || (ranks == 0 && cu_seqlens == nullptr) ||
      (ranks > 0 && page_table == nullptr) || (page_table != nullptr && (slots == nullptr || kv_lens == nullptr)))
    return LRM_BAD_ARGUMENT;
  if (!lrm_attention_gated_supports(d, dv, kTile) || out_stride % 2 != 0 || reinterpret_cast<uintptr_t>(out) % 4 != 0 ||
      (reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) % 16 != 0)
    return LRM_UNSUPPORTED;
  const Source src{k, v, page_table, table_stride, slots, kv_lens};
  const Geometry g{seqs, max_seq_len, q_heads, kv_heads, d, dv, ranks, Fresh{}};
  if (ranks > 0) LRM_BY_SIZES(launch_decode);
  LRM_BY_SIZES(launch_tiled);
}

// The decode step from the float32 projection on: proj [seqs, stride] holds rows [q_heads * d | kv_heads * d |
// kv_heads * dv] (`gate`, where there is one, usually their further columns). bias float32 [row] or null; table float32
// [seqs, rotary / 2, 2] (null with rotary 0); the new key and value go to rows dest_rows [seqs] of the pages.
LRM_API int lrm_attention_gated_decode_fused(const float* proj, long long stride, const float* bias, const float* table,
                                             int rotary, void* k_pages, void* v_pages, const int* dest_rows,
                                             const int* page_table, int table_stride, const int* slots, const int* kv_lens,
                                             int seqs, int q_heads, int kv_heads, int d, int dv, float scale, float cap,
                                             int window, int keep, const float* sinks, const float* gate,
                                             long long gate_stride, int gate_per_head, void* out, long long out_stride,
                                             float out_scale, int ranks, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  const Form f = make_form(scale, cap, window, keep, sinks, gate, gate_stride, gate_per_head, out, out_stride, out_scale);
  if (bad_form(f, q_heads, kv_heads, d, dv) || ranks < 1 || ranks > kMaxRanks || proj == nullptr || dest_rows == nullptr ||
      page_table == nullptr || slots == nullptr || kv_lens == nullptr || rotary < 0 || rotary % 2 || rotary > d ||
      (rotary > 0 && table == nullptr) || stride < q_heads * d + static_cast<long long>(kv_heads) * (d + dv))
    return LRM_BAD_ARGUMENT;
  if (!lrm_attention_gated_supports(d, dv, kTile) || out_stride % 2 != 0 || reinterpret_cast<uintptr_t>(out) % 4 != 0 ||
      (reinterpret_cast<uintptr_t>(k_pages) | reinterpret_cast<uintptr_t>(v_pages)) % 16 != 0)
    return LRM_UNSUPPORTED;
  const Source src{k_pages, v_pages, page_table, table_stride, slots, kv_lens};
  const Geometry g{seqs, 1, q_heads, kv_heads, d, dv, ranks,
                   Fresh{proj, stride, bias, reinterpret_cast<const float2*>(table), rotary, dest_rows}};
  const void* q = nullptr;
  const int* cu_seqlens = nullptr;
  LRM_BY_SIZES(launch_decode);
}
