// Gated softmax attention (the form of attention_gated.cu: a cap on the scores, sinks, a window or a chunk beside
// kept first keys, an output gate, values of their own width) for prompts on the 5th-generation tensor cores,
// from the step's packed bfloat16 q, k and v.
//
// One CTA = 128 queries of one head of one sequence. Keys and values arrive in tiles of 64 through TMA (128-byte
// swizzle, a ring of two stages): first the tiles of the kept keys that lie before the window, then the
// window's. For every tile
//   S = Q K^T    tcgen05.mma, M 128 x N 64, into tensor memory
//   softmax      four warps, one thread per query row: the row's largest dot product first (a score rises with
//                its dot product, so the map to capped scores is applied to the maximum alone), then
//                P = 2^(s - m), rounded to bfloat16 and written over the scores it came from
//   O += P V     tcgen05.mma with P from tensor memory as the A operand and V MN-major from shared memory
// O stays in tensor memory and is rescaled only when a row's maximum has moved by more than 2^8 since the scale
// O was last brought to. A sink is where a row's maximum and mass begin. Several CTAs per SM take turns on the
// tensor core. At the end a thread divides its row by the mass, multiplies it by its gates and stores it.
//
// Head sizes are multiples of 8 up to 128. The tensor maps have three dimensions (column of a head, head, token):
// boxes of 64 columns that reach beyond a head read zeros there, so heads of any such size fill whole
// swizzled blocks. Rows and keys outside a sequence are zeros or a neighbour's; the mask hides such keys and such
// rows are never stored. Every mbarrier wait is bounded; a wait that gives up records a code in `status`, and the
// CTA winds down and frees its tensor memory. No cluster multicast.
#include "attention_gated.cuh"
#include "umma.cuh"

namespace {

constexpr int BQ = 128, BKV = kKeyTile, UMMA_K = 16, STAGES = 2;
constexpr int kLoaderWarp = 4, kIssuerWarp = 5, kGatedThreads = 6 * 32;
constexpr float kRescaleStep = 8.0f;  // log2: O is rescaled when the maximum moved this far

enum : int { kStuckQ = 41, kStuckKV = 42, kStuckScores = 43, kStuckProbabilities = 44, kStuckOutput = 45,
             kStuckStage = 46, kMisaligned = 47 };

__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* map, uint64_t* bar, int x, int y, int z) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
      ::"r"(smem_u32(dst)), "l"(reinterpret_cast<uint64_t>(map)), "r"(smem_u32(bar)), "r"(x), "r"(y), "r"(z)
      : "memory");
}

// One chunk of 32 scores of a row -> probabilities packed in pairs; `edge` tiles test every key.
template <bool CAPPED, bool EDGE>
__device__ __forceinline__ float probabilities(const uint32_t (&s)[32], uint32_t (&packed)[16], const ScoreMap& map,
                                               const Form& f, float m_use, int key0, int row, int row_first) {
  float sum = 0.f;
#pragma unroll
  for (int e = 0; e < 32; e += 2) {
    float p[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const float dot = __uint_as_float(s[e + u]);
      p[u] = unit_exp2(CAPPED ? map.cap(dot) - m_use : fmaf(dot, map.mul, -m_use));
      if (EDGE && !sees(f, key0 + e + u, row, row_first)) p[u] = 0.f;
    }
    sum += p[0] + p[1];
    packed[e >> 1] = pack_bf16(p[0], p[1]);
  }
  return sum;
}

// Shared memory (1024-byte aligned): Q [128][DK] | stages of (K [64][DK] | V [64][DV]) | barriers; a tile is
// one or two blocks of 64 columns (a swizzle row is 128 bytes), one after the other.
template <int DK, int DV, int CTAS>
__global__ __launch_bounds__(kGatedThreads, CTAS) void gated_umma_kernel(
    const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
    const __grid_constant__ CUtensorMap map_v, Form f, const int* __restrict__ cu_seqlens, int q_heads, int kv_heads,
    int d, int dv, int* __restrict__ status) {
  constexpr uint32_t Q_BLOCK = BQ * 64 * 2, Q_TILE = Q_BLOCK * (DK / 64);
  constexpr uint32_t KV_BLOCK = BKV * 64 * 2, K_TILE = KV_BLOCK * (DK / 64), V_TILE = KV_BLOCK * (DV / 64);
  constexpr uint32_t STAGE = K_TILE + V_TILE;
  constexpr uint32_t kTmemColumns = BKV + DV <= 128 ? 128 : 256;  // a power of two
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  if ((smem_u32(smem_raw) & 1023u) != 0) {  // the swizzled tiles need it; give up rather than compute nonsense
    if (threadIdx.x == 0 && status != nullptr) atomicCAS(status, 0, kMisaligned);
    return;
  }
  unsigned char* q_tile = smem_raw;
  unsigned char* kv_tiles = q_tile + Q_TILE;  // stage s: K at s * STAGE, V right after
  uint64_t* q_full = reinterpret_cast<uint64_t*>(kv_tiles + STAGES * STAGE);
  uint64_t* kv_full = q_full + 1;             // [STAGES]
  uint64_t* kv_free = kv_full + STAGES;       // [STAGES]
  uint64_t* s_full = kv_free + STAGES;        // scores written
  uint64_t* p_ready = s_full + 1;             // probabilities written (4 warps arrive)
  uint64_t* o_done = p_ready + 1;             // the last P V is complete
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 1);
  volatile int* bail = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int qt = gridDim.z - 1 - blockIdx.z;  // the longest rows of work first
  const int h = blockIdx.x, b = blockIdx.y;
  const int start = cu_seqlens[b], len = cu_seqlens[b + 1] - start;
  const int q0 = qt * BQ;
  if (q0 >= len) return;
  const int kh = h / (q_heads / kv_heads);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int first_key = first_visible_key(q0, f.window);
  const Tiles tiles(first_key, min(q0 + BQ, len) - 1, f.keep);

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(kv_full + s, 1);
      mbar_init(kv_free + s, 1);
    }
    mbar_init(s_full, 1);
    mbar_init(p_ready, 4);
    mbar_init(o_done, 1);
    *bail = 0;
    mbar_fence_init();
  }
  if (warp == kIssuerWarp) {
    tmem_alloc(tmem_slot, kTmemColumns);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + BKV;
  // Barriers and tensor memory were set up while the kernel that produces q, k and v may still have been
  // running (sequence bounds are the step's own input); its results are read from here on.
  pdl_wait();

  if (warp == kLoaderWarp) {
    if (lane == 0) {
      // ---- one thread brings the query tile once and the key and value tiles through the ring
      mbar_expect_tx(q_full, Q_TILE);
#pragma unroll
      for (int db = 0; db < DK / 64; ++db) tma_load_3d(q_tile + db * Q_BLOCK, &map_q, q_full, db * 64, h, start + q0);
      int issued = 0;
      for (; issued < tiles.count && !*bail; ++issued) {
        const int s = issued % STAGES;
        if (issued >= STAGES && !mbar_wait(kv_free + s, ((issued / STAGES) - 1) & 1, status, kStuckStage)) {
          *bail = 1;
          break;
        }
        const int row = start + tiles.at(issued) * BKV;
        unsigned char* kdst = kv_tiles + s * STAGE;
        mbar_expect_tx(kv_full + s, STAGE);
#pragma unroll
        for (int db = 0; db < DK / 64; ++db) tma_load_3d(kdst + db * KV_BLOCK, &map_k, kv_full + s, db * 64, kh, row);
#pragma unroll
        for (int db = 0; db < DV / 64; ++db)
          tma_load_3d(kdst + K_TILE + db * KV_BLOCK, &map_v, kv_full + s, db * 64, kh, row);
      }
      if (*bail) {  // wait (bounded) for the copies already in flight before the CTA may exit
        mbar_wait(q_full, 0, status, kStuckQ);
        for (int i = issued > STAGES ? issued - STAGES : 0; i < issued; ++i)
          mbar_wait(kv_full + i % STAGES, (i / STAGES) & 1, status, kStuckKV);
      }
    }
  } else if (warp == kIssuerWarp) {
    if (lane == 0) {
      // ---- one thread drives the tensor core
      constexpr uint32_t idesc_s = umma_idesc(BQ, BKV);        // both K-major
      constexpr uint32_t idesc_pv = umma_idesc(BQ, DV, true);  // V is MN-major
      auto scores = [&](int j) {  // S = Q K_j^T
        const uint32_t qa = smem_u32(q_tile), ka = smem_u32(kv_tiles + (j % STAGES) * STAGE);
#pragma unroll
        for (int k = 0; k < DK / UMMA_K; ++k) {  // 64-column block, then 32 bytes per step
          if (k * UMMA_K >= d) break;            // columns beyond the head are zeros on both sides
          const uint32_t step = (k % 4) * UMMA_K * 2;
          umma_bf16(tmem_s, smem_desc(qa + (k / 4) * Q_BLOCK + step), smem_desc(ka + (k / 4) * KV_BLOCK + step), idesc_s,
                    k > 0 ? 1u : 0u);
        }
        umma_commit(s_full);
      };
      bool ok = mbar_wait(q_full, 0, status, kStuckQ) && mbar_wait(kv_full, 0, status, kStuckKV);
      if (ok) {
        tc_fence_after();
        scores(0);
      }
      for (int j = 0; j < tiles.count && ok; ++j) {
        ok = mbar_wait(p_ready, j & 1, status, kStuckProbabilities);
        if (!ok) break;
        tc_fence_after();
        const uint32_t va = smem_u32(kv_tiles + (j % STAGES) * STAGE + K_TILE);
#pragma unroll
        for (int k = 0; k < BKV / UMMA_K; ++k)  // O (+)= P V_j, P from tensor memory (8 columns per 16 keys)
          umma_bf16_a_tmem(tmem_o, tmem_s + k * (UMMA_K / 2), smem_desc(va + k * UMMA_K * 128, KV_BLOCK), idesc_pv,
                           (j > 0 || k > 0) ? 1u : 0u);
        umma_commit(kv_free + j % STAGES);  // every product that reads stage j has been issued
        if (j + 1 == tiles.count) {
          umma_commit(o_done);
          break;
        }
        ok = mbar_wait(kv_full + (j + 1) % STAGES, ((j + 1) / STAGES) & 1, status, kStuckKV);
        if (!ok) break;
        tc_fence_after();
        scores(j + 1);
      }
      if (!ok) *bail = 1;
    }
  } else {
    // ---- softmax and output: one thread per query row; a warp may touch the quarter of the tensor memory's
    // lanes given by its index
    const int row = q0 + warp * 32 + lane;  // position in the sequence
    const uint32_t lane_base = static_cast<uint32_t>(warp * 32) << 16;
    const uint32_t my_s = tmem_s + lane_base, my_o = tmem_o + lane_base;
    const ScoreMap map(f);
    const int row_first = first_visible_key(row, f.window);
    const int whole_from = first_visible_key(q0 + BQ - 1, f.window);
    const float sink_log2 = f.sinks != nullptr ? f.sinks[h] * kLog2e : -INFINITY;
    // the row's gates are wanted at the end: have them in L2 by then
    const size_t tok = static_cast<size_t>(start + min(row, len - 1));
    const bool by_element = f.gate != nullptr && !f.gate_per_head;
    const float* gates = by_element ? f.gate + tok * f.gate_stride + h * dv : nullptr;
    if (by_element)
      for (int c = 0; c < dv; c += 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(gates + c));
    float m_run = sink_log2;   // the row's true running maximum (log2 domain)
    float m_ref = -INFINITY;   // the maximum O and the mass are scaled by
    float l = 0.f;
    bool ok = true;
    for (int j = 0; j < tiles.count; ++j) {
      const bool here = !*bail && mbar_wait(s_full, j & 1, status, kStuckScores);
      if (!__all_sync(0xffffffffu, here)) {  // the warp leaves together
        *bail = 1;
        ok = false;
        break;
      }
      tc_fence_after();
      const int key0 = tiles.at(j) * BKV;
      // tiles all of whose keys every query of the CTA sees need no test per score
      const bool edge = key0 + BKV - 1 > q0 || (key0 < whole_from && key0 + BKV > f.keep);
      // pass 1: the row's largest dot product in this tile
      float mx = -INFINITY;
      {
        uint32_t sc[BKV / 32][32];
#pragma unroll
        for (int c = 0; c < BKV / 32; ++c) tmem_load32_async(my_s + c * 32, sc[c]);
        tmem_load_wait();
#pragma unroll
        for (int c = 0; c < BKV / 32; ++c) tmem_pin(sc[c]);
        if (edge) {
#pragma unroll
          for (int c = 0; c < BKV / 32; ++c)
#pragma unroll
            for (int e = 0; e < 32; ++e)
              if (sees(f, key0 + c * 32 + e, row, row_first)) mx = fmaxf(mx, __uint_as_float(sc[c][e]));
        } else {
#pragma unroll
          for (int c = 0; c < BKV / 32; ++c)
#pragma unroll
            for (int e = 0; e < 32; ++e) mx = fmaxf(mx, __uint_as_float(sc[c][e]));
        }
      }
      if (mx > -INFINITY) m_run = fmaxf(m_run, map.capped ? map.cap(mx) : map.plain(mx));
      // bring O and the mass to the new maximum only when it has moved far (for the first tile, where O
      // holds nothing yet, only the reference is set and a sink's share of the mass with it)
      const bool far = m_run > m_ref + kRescaleStep;
      if (j == 0) {
        m_ref = m_run;
        if (f.sinks != nullptr) l = unit_exp2(sink_log2 - m_ref);
      } else if (__any_sync(0xffffffffu, far)) {
        const float alpha = far ? unit_exp2(m_ref - m_run) : 1.0f;  // m_ref = -inf gives 0, and O is 0 then
#pragma unroll 1
        for (int c = 0; c < DV / 32; ++c) {
          uint32_t r[32];
          tmem_load32(my_o + c * 32, r);
#pragma unroll
          for (int e = 0; e < 32; ++e) r[e] = __float_as_uint(__uint_as_float(r[e]) * alpha);
          tmem_store32(my_o + c * 32, r);
        }
        tmem_store_wait();
        l *= alpha;
        if (far) m_ref = m_run;
      }
      const float m_use = m_ref == -INFINITY ? 0.f : m_ref;  // a row that has seen no key yet
      // pass 2: probabilities against m_ref, written over the scores they came from: keys 32 c .. 32 c + 31
      // become columns 16 c .. 16 c + 15 (read by then)
      float sum = 0.f;
      uint32_t sc[BKV / 32][32];
      tmem_load32_async(my_s, sc[0]);
#pragma unroll
      for (int c = 0; c < BKV / 32; ++c) {
        tmem_load_wait();
        tmem_pin(sc[c]);
        if (c + 1 < BKV / 32) tmem_load32_async(my_s + (c + 1) * 32, sc[c + 1]);
        uint32_t packed[16];
        const int at = key0 + c * 32;
        if (map.capped)
          sum += edge ? probabilities<true, true>(sc[c], packed, map, f, m_use, at, row, row_first)
                      : probabilities<true, false>(sc[c], packed, map, f, m_use, at, row, row_first);
        else
          sum += edge ? probabilities<false, true>(sc[c], packed, map, f, m_use, at, row, row_first)
                      : probabilities<false, false>(sc[c], packed, map, f, m_use, at, row, row_first);
        tmem_store16(my_s + c * 16, packed);
      }
      tmem_store_wait();
      l += sum;
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
    }
    // 32 gates at a time on the way into registers, the first ones while the last product runs
    const bool fours = by_element && f.gate_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(f.gate) & 15) == 0 && dv % 4 == 0;
    float z[32];
    auto load_gates = [&](int c) {
      if (!by_element) return;
#pragma unroll
      for (int e = 0; e < 32; e += 4) {
        if (c + e >= dv) break;  // (dv is a multiple of 8)
        if (fours) {
          const float4 four = *reinterpret_cast<const float4*>(gates + c + e);
          z[e] = four.x, z[e + 1] = four.y, z[e + 2] = four.z, z[e + 3] = four.w;
        } else {
#pragma unroll
          for (int u = 0; u < 4; ++u) z[e + u] = gates[c + e + u];
        }
      }
    };
    load_gates(0);
    if (ok && !__all_sync(0xffffffffu, mbar_wait(o_done, 0, status, kStuckOutput))) {
      *bail = 1;
      ok = false;
    }
    tc_fence_after();
    if (ok) {
      // the mass belongs to m_ref, and so does O: their quotient is the row's attention
      const float factor = (by_element ? f.out_scale : gate_at(f, tok, h, dv, 0)) / l;
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(f.out) + tok * f.out_stride + h * dv;
#pragma unroll 1
      for (int c = 0; c < dv; c += 32) {
        uint32_t r[32];
        tmem_load32(my_o + c, r);
        if (row < len) {
#pragma unroll
          for (int e = 0; e < 32; e += 8) {
            if (c + e >= dv) break;
            uint32_t packed[4];
#pragma unroll
            for (int u = 0; u < 8; u += 2) {
              float x = __uint_as_float(r[e + u]) * factor, y = __uint_as_float(r[e + u + 1]) * factor;
              if (by_element) {
                x *= unit_sigmoid(z[e + u]);
                y *= unit_sigmoid(z[e + u + 1]);
              }
              packed[u >> 1] = pack_bf16(x, y);
            }
            *reinterpret_cast<uint4*>(dst + c + e) = make_uint4(packed[0], packed[1], packed[2], packed[3]);
          }
        }
        load_gates(c + 32);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == kIssuerWarp) tmem_dealloc(tmem_s, kTmemColumns);
}

// [tokens, heads, d] bfloat16, boxes of `box_rows` tokens x 64 columns of one head, zeros beyond the head.
bool make_head_map(CUtensorMap* map, const void* base, long long tokens, int heads, int d, int box_rows) {
  EncodeTiledFn fn = encode_tiled();
  if (fn == nullptr) return false;
  const cuuint64_t dims[3] = {static_cast<cuuint64_t>(d), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(tokens)};
  const cuuint64_t strides[2] = {static_cast<cuuint64_t>(d) * 2, static_cast<cuuint64_t>(d) * heads * 2};
  const cuuint32_t box[3] = {64, 1, static_cast<cuuint32_t>(box_rows)};
  const cuuint32_t elem[3] = {1, 1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, elem,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int DK, int DV, int CTAS>
int launch(const void* q, const void* k, const void* v, const Form& f, const int* cu_seqlens, int tokens, int seqs,
           int max_seq_len, int q_heads, int kv_heads, int d, int dv, int* status, cudaStream_t stream) {
  CUtensorMap map_q, map_k, map_v;
  if (!make_head_map(&map_q, q, tokens, q_heads, d, BQ) || !make_head_map(&map_k, k, tokens, kv_heads, d, BKV) ||
      !make_head_map(&map_v, v, tokens, kv_heads, dv, BKV))
    return LRM_UNSUPPORTED;
  constexpr int smem = BQ * DK * 2 + STAGES * BKV * (DK + DV) * 2 + 256;
  auto kernel = gated_umma_kernel<DK, DV, CTAS>;
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return static_cast<int>(e);
  const int q_tiles = (max_seq_len + BQ - 1) / BQ;
  if (seqs > 65535 || q_tiles > 65535) return LRM_UNSUPPORTED;
  LRM_LAUNCH(kernel, dim3(q_heads, seqs, q_tiles), kGatedThreads, smem, stream, map_q, map_k, map_v, f, cu_seqlens,
             q_heads, kv_heads, d, dv, status);
  return 0;
}

}  // namespace

// 1 when the kernel takes these head sizes: multiples of 8 (TMA wants pitches of 16 bytes) up to 128.
LRM_API int lrm_attention_gated_umma_supports(int d, int dv) {
  return d > 0 && dv > 0 && d <= 128 && dv <= 128 && d % 8 == 0 && dv % 8 == 0 && encode_tiled() != nullptr ? 1 : 0;
}

// q [tokens, q_heads, d], k, v [tokens, kv_heads, d | dv] packed bfloat16 of prompts (sequence b: rows cu_seqlens[b] ..
// cu_seqlens[b + 1] - 1, at most max_seq_len of them), 16-byte aligned; out bfloat16 (pointer at its first column),
// rows out_stride elements apart, both on 16-byte boundaries; scale positive; the rest as for lrm_attention_gated.
// `status`: one int in device memory, 0 before the launch; a kernel that gave up on a wait writes a code there.
LRM_API int lrm_attention_gated_umma(const void* q, const void* k, const void* v, const int* cu_seqlens, int tokens, int seqs,
                                     int max_seq_len, int q_heads, int kv_heads, int d, int dv, float scale, float cap,
                                     int window, int keep, const float* sinks, const float* gate, long long gate_stride,
                                     int gate_per_head, void* out, long long out_stride, float out_scale, int* status,
                                     cudaStream_t stream) {
  if (seqs <= 0 || max_seq_len <= 0 || tokens <= 0) return 0;
  const Form f = make_form(scale, cap, window, keep, sinks, gate, gate_stride, gate_per_head, out, out_stride, out_scale);
  if (bad_form(f, q_heads, kv_heads, d, dv) || cu_seqlens == nullptr || status == nullptr || !(scale > 0.f))
    return LRM_BAD_ARGUMENT;
  if (!lrm_attention_gated_umma_supports(d, dv) || q_heads > 65535 || out_stride % 8 != 0 ||
      (reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) |
       reinterpret_cast<uintptr_t>(out)) % 16 != 0)
    return LRM_UNSUPPORTED;
#define LRM_GATED(DIM, VDIM, CTAS) \
  launch<DIM, VDIM, CTAS>(q, k, v, f, cu_seqlens, tokens, seqs, max_seq_len, q_heads, kv_heads, d, dv, status, stream)
  if (d <= 64) return dv <= 64 ? LRM_GATED(64, 64, 3) : LRM_GATED(64, 128, 2);
  return dv <= 64 ? LRM_GATED(128, 64, 2) : LRM_GATED(128, 128, 2);
#undef LRM_GATED
}
