"""Which attention kernel runs for a geometry.

The row-wise kernel (csrc/attention_rowwise.cu) takes every head size up to
512 and both dtypes, and is the only attention of the float32 path. bfloat16
prompts with head size 64 or 128 run the TMA + tcgen05 kernel
(csrc/attention_prefill_umma.cu); bfloat16 with head size 32, 64 or 128 and
64-token pages otherwise runs the warp-level tiled kernels (csrc/attention_tiled.cu).
A bfloat16 decode step of a layer that writes its own unwindowed cache runs rotation,
cache write, attention and the merge of the splits as one cluster kernel
(csrc/attention_decode_cluster.cu). A step that appends several tokens to started
sequences stores its keys first and attends over the cache (row-wise, or the tiled
extend kernel in bfloat16). bfloat16 attention over one key head whose rows also hold the
values (latent attention's cache) runs csrc/attention_shared_keys.cu in every phase.
Attention without a softmax (a key's weight is the sigmoid of its score) has kernels of its own in
csrc/attention_sigmoid.cu: tiled in bfloat16 for head sizes 32, 64, 96 and 128, row-wise otherwise.
Softmax attention with a cap on its scores, kept first keys or an output gate (and then also with sinks and
values of another width) runs csrc/attention_gated.cu: tiled in bfloat16 for head sizes that are multiples of
8 up to 128 (prompts on tcgen05, csrc/attention_gated_umma.cu), row-wise otherwise.

`attend` is the one call a mixer makes: it takes the step's projection and picks
rotation, cache write and attention kernels for the step's phase and geometry.
"""
from __future__ import annotations

import ctypes
import os
from dataclasses import dataclass
from typing import Optional

import torch

from . import library
from .ops import _code, _done, _ptr, _stream  # noqa: PLC2701

SM_COUNT = 148
force_rowwise = False  # tests switch the tiled kernels off to compare both paths
force_warp_level = False  # tests keep prompts off the tcgen05 kernel to cover the warp-level one
force_unfused_decode = False  # tests keep decode steps on the separate rotation / attention / merge kernels
force_cluster_size = None  # tests fix the CTAs per cluster of the fused decode kernel
force_shared_key_splits = None  # tests fix the splits of the shared-key kernel's decode step
force_sigmoid_ranks = None  # tests fix the CTAs per cluster of the sigmoid decode kernel
force_gated_split = False  # tests keep decode steps of that kernel behind a split of the projection in its own launch
force_gated_ranks = None  # tests fix the CTAs per cluster of the gated softmax kernel's decode step
prefill_kernel = None  # tests pin the tcgen05 prompt kernel: "pingpong" or "single" (None: the rule in prefill())


@dataclass(frozen=True)
class Extras:
    """What some attention layers have beyond the plain softmax over scaled scores.

    sinks: float32 [query heads]; exp(sink_h) is added to the softmax's denominator (a key that
        is always seen, has no value, and whose score is not scaled).
    temperature: (coef, every); the query at position p counts 1 + coef * ln(floor((p + 1) / every)
        + 1) times. The kernels put the factor into the score's scale, in float32.
    """

    sinks: Optional[torch.Tensor] = None
    temperature: Optional[tuple] = None

    @property
    def plain(self) -> bool:
        return self.sinks is None and self.temperature is None

    def arguments(self):
        """(sinks pointer, coef, every) as the kernels take them."""
        coef, every = self.temperature if self.temperature is not None else (0.0, 0)
        return _ptr(self.sinks), ctypes.c_float(coef), int(every)


NO_EXTRAS = Extras()


@dataclass(frozen=True)
class Shaping:
    """What some attention layers do to their queries and keys between the projection and the
    attention itself (csrc/shaped_qkv.cu applies it in this order, each step only if given).

    taps: float32 [n, projection row], a causal convolution over time on every projected channel,
        with `tails`, the StateView of the sequences' last n - 1 unbiased projections.
    row_norm: (q weight, k weight), an RMS norm over all query columns and one over all key columns
        (eps `row_eps`).
    inv_freq, rotary, adjacent_pairs: a rotation of each head's first `rotary` dimensions, angle =
        position * inv_freq[i] (float64 [rotary / 2]), cosines and sines times `magnitude`; dimension i
        pairs with i + rotary / 2, or 2i with 2i + 1.
    head_weights: (q weight, k weight), an RMS norm over every query and every key head ahead of the
        rotation, one weight of the head size each (eps `head_weight_eps`).
    head_norm_eps: each query and key head is divided by its root mean square afterwards.
    """

    taps: Optional[torch.Tensor] = None
    tails: Optional[object] = None
    row_norm: Optional[tuple] = None
    row_eps: float = 0.0
    head_weights: Optional[tuple] = None
    head_weight_eps: float = 0.0
    inv_freq: Optional[torch.Tensor] = None
    magnitude: float = 1.0
    rotary: int = 0
    adjacent_pairs: bool = False
    head_norm_eps: Optional[float] = None


def _value_stride(kv) -> int:
    """Elements between two value rows of a cache view: values that live inside the key rows are
    read from the keys' storage with the keys' width."""
    return kv.k.shape[3] if getattr(kv, "values_in_keys", False) else kv.v.shape[3]


def _shared_keys(q, kv_heads: int, dv: int, slopes, out_scale: float, extras) -> bool:
    """True when the kernel for one key head whose rows hold the values (latent attention's cache
    layout, csrc/attention_shared_keys.cu) takes this attention; it knows sinks, not the temperature."""
    return (not force_rowwise and q.dtype == torch.bfloat16 and kv_heads == 1 and slopes is None
            and out_scale == 1.0 and extras.temperature is None and q.data_ptr() % 16 == 0
            and bool(library.load().lrm_attention_shared_keys_supports(q.shape[1], q.shape[2], dv, 64)))


def _tiled(q, page_size: int) -> bool:
    return (not force_rowwise and q.dtype == torch.bfloat16
            and bool(library.load().lrm_attention_tiled_supports(q.shape[2], page_size)))


def _plain(q, dv: int, slopes, out_scale: float) -> bool:
    """True for attention as the tensor-core kernels compute it: values as wide as keys, no
    distance penalty, the result not scaled."""
    return dv == q.shape[2] and slopes is None and out_scale == 1.0


def prefill(q, k, v, out, cu_seqlens, seq_of_token, max_seq_len: int, scale: float, window: int,
            slopes=None, out_scale: float = 1.0, extras=None, value_dim=None) -> None:
    """`v` None: the values are the first `value_dim` columns of the key rows."""
    T, Hq, d = q.shape
    extras = extras or NO_EXTRAS
    lib = library.load()
    if v is None or not extras.plain:
        dv = value_dim if v is None else v.shape[2]
        shared = v is None or v.data_ptr() == k.data_ptr()
        if shared and dv != d and k.data_ptr() % 16 == 0 and _shared_keys(q, k.shape[1], dv, slopes, out_scale, extras):
            _done(lib.lrm_attention_shared_keys(_ptr(q), _ptr(k), None, _ptr(out), _ptr(cu_seqlens), None, None, 0,
                                                None, cu_seqlens.numel() - 1, max_seq_len, Hq, d, dv,
                                                ctypes.c_float(scale), window, None, 1, _ptr(extras.sinks), _stream()),
                  "attention_shared_keys")
            return
        if dv == d and _tiled(q, 64) and shared:
            _done(lib.lrm_attention_prefill_tiled(_ptr(q), _ptr(k), _ptr(k), _ptr(out), _ptr(cu_seqlens),
                                                  cu_seqlens.numel() - 1, max_seq_len, Hq, k.shape[1], d,
                                                  ctypes.c_float(scale), window, _ptr(slopes),
                                                  ctypes.c_float(out_scale), *extras.arguments(), _stream()),
                  "attention_prefill_tiled")
            return
        _done(lib.lrm_attention_packed_rowwise(_ptr(q), _ptr(k), _ptr(k if v is None else v), _ptr(out),
                                               _code(q.dtype), _ptr(cu_seqlens), _ptr(seq_of_token), T, Hq,
                                               k.shape[1], d, dv, ctypes.c_float(scale), window, _ptr(slopes),
                                               ctypes.c_float(out_scale), *extras.arguments(),
                                               d if v is None else dv, _stream()),
              "attention_packed_rowwise")
        return
    dv = v.shape[2]
    aligned = all(t.data_ptr() % 16 == 0 for t in (q, k, v, out))
    if (not force_rowwise and not force_warp_level and q.dtype == torch.bfloat16 and aligned and window >= 0
            and _plain(q, dv, slopes, out_scale) and lib.lrm_attention_prefill_umma_supports(d)):
        from . import gemm_dispatch
        gemm_dispatch.mark_status_dirty()
        # Two tcgen05 kernels. The one that keeps probabilities and output in tensor memory wins on
        # long prompts and on batches of prompts: at head size 128 (one query tile per CTA on key tiles
        # of 64 up to 2,304 tokens, two query tiles taking turns beyond) from 1,536 tokens on (2,048
        # tokens 60 against 86 us, 953 against 582 TFLOP/s at 32,768); at head size 64 (four CTAs per SM on key tiles of 64) beyond 2,048 tokens (3,072
        # tokens 78 against 100 us, 681 against 534 TFLOP/s at 32,768) and whenever several prompts
        # are packed (four of 512 tokens 20 against 29 us, eight of 128 tokens 9.5 against 11.1). A
        # single short prompt is bound by the chain of key tiles of its last query tile, which the
        # older kernel, with two threads per row, walks a little faster (1,024 tokens 24 against 26 us).
        # Packed prompts go to the newer kernel at head size 128 too (four of 512 tokens 33 against 46 us).
        # (several prompts: the packed tokens are well more than the longest prompt; a short prompt
        # filled up to whole rows with a few tokens of padding does not count)
        pingpong = (max_seq_len >= 1536 if d == 128 else max_seq_len > 2048) or 4 * T >= 5 * max_seq_len
        if prefill_kernel is not None:
            pingpong = prefill_kernel == "pingpong"
        if pingpong:
            _done(lib.lrm_attention_prefill_pingpong(_ptr(q), _ptr(k), _ptr(v), _ptr(out), _ptr(cu_seqlens), T,
                                                     cu_seqlens.numel() - 1, max_seq_len, Hq, k.shape[1], d,
                                                     ctypes.c_float(scale), window,
                                                     _ptr(gemm_dispatch._status_word(q.device)), _stream()),
                  "attention_prefill_pingpong")
            return
        _done(lib.lrm_attention_prefill_umma(_ptr(q), _ptr(k), _ptr(v), _ptr(out), _ptr(cu_seqlens), T,
                                             cu_seqlens.numel() - 1, max_seq_len, Hq, k.shape[1], d,
                                             ctypes.c_float(scale), window,
                                             _ptr(gemm_dispatch._status_word(q.device)), _stream()),
              "attention_prefill_umma")
        return
    if dv == d and _tiled(q, 64):
        _done(lib.lrm_attention_prefill_tiled(_ptr(q), _ptr(k), _ptr(v), _ptr(out), _ptr(cu_seqlens),
                                              cu_seqlens.numel() - 1, max_seq_len, Hq, k.shape[1], d,
                                              ctypes.c_float(scale), window, _ptr(slopes),
                                              ctypes.c_float(out_scale), *NO_EXTRAS.arguments(), _stream()),
              "attention_prefill_tiled")
        return
    _done(lib.lrm_attention_packed_rowwise(_ptr(q), _ptr(k), _ptr(v), _ptr(out), _code(q.dtype),
                                           _ptr(cu_seqlens), _ptr(seq_of_token), T, Hq, k.shape[1], d, dv,
                                           ctypes.c_float(scale), window, _ptr(slopes),
                                           ctypes.c_float(out_scale), *NO_EXTRAS.arguments(), dv, _stream()),
          "attention_packed_rowwise")


CTAS_PER_SM = 4  # decode attention CTAs wanted per SM (each keeps one 64-key K/V tile in flight)


def decode_splits(seqs: int, kv_heads: int, group: int, max_kv_len: int, window: int) -> int:
    """Splits of the key range so that about CTAS_PER_SM CTAs per SM stream the cache."""
    ctas = seqs * kv_heads * -(-group // 16)
    keys = min(max_kv_len, abs(window) + 63) if window else max_kv_len  # a chunk (window < 0) shows no more either
    pages = max(1, -(-keys // 64))
    return max(1, min(pages, -(-CTAS_PER_SM * SM_COUNT // ctas)))


def decode(q, kv, out, slots, kv_lens, max_kv_len: int, scale: float, window: int,
           slopes=None, out_scale: float = 1.0, extras=None) -> None:
    from .ops import _value_dim
    B, Hq, d = q.shape
    dv = _value_dim(kv)
    extras = extras or NO_EXTRAS
    lib = library.load()
    if (getattr(kv, "values_in_keys", False) and dv != d and kv.page_size == 64
            and _shared_keys(q, kv.kv_heads, dv, slopes, out_scale, extras)):
        # few CTAs (sequences x groups of 32 heads): the key tiles are cut until the SMs are filled once
        # with as many CTAs as their shared memory lets run side by side (two at key width 288, one at
        # 544); more splits than that only add a second wave of CTAs and partial rows for the merge
        keys = min(max_kv_len, window + 63) if window > 0 else max_kv_len
        room = int(lib.lrm_attention_shared_keys_ctas_per_sm(d)) * SM_COUNT
        splits = max(1, min(-(-keys // 64), room // (B * -(-Hq // 32))))
        if force_shared_key_splits is not None:
            splits = force_shared_key_splits
        partials = torch.empty((B, Hq, splits, dv + 2), dtype=torch.float32, device=q.device) if splits > 1 else None
        _done(lib.lrm_attention_shared_keys(_ptr(q), None, _ptr(kv.k), _ptr(out), None, _ptr(kv_lens),
                                            _ptr(kv.page_table), kv.page_table.shape[1], _ptr(slots), B, 1, Hq, d,
                                            dv, ctypes.c_float(scale), window, _ptr(partials), splits, _ptr(extras.sinks),
                                            _stream()),
              "attention_shared_keys", launches=2 if splits > 1 else 1)
        return
    if dv == d and _tiled(q, kv.page_size):
        splits = decode_splits(B, kv.kv_heads, Hq // kv.kv_heads, max_kv_len, window)
        partials = torch.empty((B, Hq, splits, d + 2), dtype=torch.float32, device=q.device)
        _done(lib.lrm_attention_decode_tiled(_ptr(q), _ptr(kv.k), _ptr(kv.v), _ptr(partials), _ptr(out),
                                             _ptr(kv.page_table), kv.page_table.shape[1], _ptr(slots),
                                             _ptr(kv_lens), B, Hq, kv.kv_heads, d, kv.page_size,
                                             ctypes.c_float(scale), window, splits, _ptr(slopes),
                                             ctypes.c_float(out_scale), *extras.arguments(), _stream()),
              "attention_decode_tiled", launches=2)
        return
    _done(lib.lrm_attention_paged_rowwise(_ptr(q), _ptr(kv.k), _ptr(kv.v), _ptr(out), _code(q.dtype),
                                          _ptr(kv.page_table), kv.page_table.shape[1], _ptr(slots),
                                          _ptr(kv_lens), None, None, B, Hq, kv.kv_heads, d, dv, kv.page_size,
                                          ctypes.c_float(scale), window, _ptr(slopes),
                                          ctypes.c_float(out_scale), *extras.arguments(), _value_stride(kv),
                                          _stream()),
          "attention_paged_rowwise")


def extend(q, kv, out, cu_seqlens, seq_of_token, positions, slots, kv_lens, max_seq_len: int, scale: float,
           window: int, slopes=None, out_scale: float = 1.0, extras=None) -> None:
    """Packed queries, several per sequence, over the cache that already holds the step's keys."""
    from .ops import _value_dim
    T, Hq, d = q.shape
    dv = _value_dim(kv)
    extras = extras or NO_EXTRAS
    lib = library.load()
    if (getattr(kv, "values_in_keys", False) and dv != d and kv.page_size == 64
            and _shared_keys(q, kv.kv_heads, dv, slopes, out_scale, extras)):
        _done(lib.lrm_attention_shared_keys(_ptr(q), None, _ptr(kv.k), _ptr(out), _ptr(cu_seqlens), _ptr(kv_lens),
                                            _ptr(kv.page_table), kv.page_table.shape[1], _ptr(slots),
                                            cu_seqlens.numel() - 1, max_seq_len, Hq, d, dv, ctypes.c_float(scale),
                                            window, None, 1, _ptr(extras.sinks), _stream()),
              "attention_shared_keys")
        return
    if dv == d and _tiled(q, kv.page_size):
        _done(lib.lrm_attention_extend_tiled(_ptr(q), _ptr(kv.k), _ptr(kv.v), _ptr(out), _ptr(cu_seqlens),
                                             _ptr(kv.page_table), kv.page_table.shape[1], _ptr(slots),
                                             _ptr(kv_lens), cu_seqlens.numel() - 1, max_seq_len, Hq,
                                             kv.kv_heads, d, kv.page_size, ctypes.c_float(scale), window,
                                             _ptr(slopes), ctypes.c_float(out_scale), *extras.arguments(),
                                             _stream()),
              "attention_extend_tiled")
        return
    # the same arithmetic, key by key in ascending order, as the packed row-wise kernel: in
    # float32 a prompt cut into portions gives the bits of the whole prompt
    _done(lib.lrm_attention_paged_rowwise(_ptr(q), _ptr(kv.k), _ptr(kv.v), _ptr(out), _code(q.dtype),
                                          _ptr(kv.page_table), kv.page_table.shape[1], _ptr(slots),
                                          _ptr(kv_lens), _ptr(seq_of_token), _ptr(positions), T, Hq,
                                          kv.kv_heads, d, dv, kv.page_size, ctypes.c_float(scale), window,
                                          _ptr(slopes), ctypes.c_float(out_scale), *extras.arguments(),
                                          _value_stride(kv), _stream()),
          "attention_paged_rowwise")


def sigmoid(q, k, v, kv, kv_heads: int, dv: int, out, out_stride: int, offset, gate, gate_stride: int, scale: float,
            window: int, out_scale: float, max_seq_len: int, max_kv_len: int, cu_seqlens, seq_of_token, positions, slots,
            kv_lens) -> None:
    """Attention with sigmoid weights (csrc/attention_sigmoid.cu): packed keys k, v, or the cache view kv
    (one query per sequence where cu_seqlens is None). `out` and `gate` are pointers at first columns."""
    T, Hq, d = q.shape
    lib = library.load()
    paged = kv is not None
    tail = (ctypes.c_float(scale), window, _ptr(offset), gate, ctypes.c_longlong(gate_stride), ctypes.c_float(out_scale))
    pages = (_ptr(kv.page_table), kv.page_table.shape[1]) if paged else (None, 0)
    keys, values = (kv.k, kv.v) if paged else (k, v)
    page_size = kv.page_size if paged else 64
    if (not force_rowwise and q.dtype == torch.bfloat16 and lib.lrm_attention_sigmoid_supports(d, dv, page_size)
            and out_stride % 2 == 0 and all(t.data_ptr() % 16 == 0 for t in (q, keys, values)) and out.value % 4 == 0):
        if paged and cu_seqlens is None:
            # the CTAs of a cluster share a sequence's pages; about two CTAs per SM, no CTA without a page
            seen = min(max_kv_len, abs(window) + 63) if window else max_kv_len
            clusters = T * kv_heads * -(-(Hq // kv_heads) // 16)
            ranks = max(1, min(8, -(-seen // 64), -(-2 * SM_COUNT // clusters)))
            if force_sigmoid_ranks is not None:
                ranks = force_sigmoid_ranks
            _done(lib.lrm_attention_sigmoid_decode(_ptr(q), _ptr(keys), _ptr(values), out, ctypes.c_longlong(out_stride),
                                                   *pages, _ptr(slots), _ptr(kv_lens), T, Hq, kv_heads, d, *tail, ranks,
                                                   _stream()), "attention_sigmoid_decode")
            return
        _done(lib.lrm_attention_sigmoid_tiled(_ptr(q), _ptr(keys), _ptr(values), out, ctypes.c_longlong(out_stride),
                                              _ptr(cu_seqlens), *pages, _ptr(slots if paged else None),
                                              _ptr(kv_lens if paged else None), cu_seqlens.numel() - 1, max_seq_len, Hq,
                                              kv_heads, d, *tail, _stream()), "attention_sigmoid_tiled")
        return
    one_each = paged and cu_seqlens is None
    _done(lib.lrm_attention_sigmoid_rowwise(_ptr(q), _ptr(keys), _ptr(values), out, _code(q.dtype),
                                            ctypes.c_longlong(out_stride), _ptr(cu_seqlens),
                                            _ptr(None if one_each else seq_of_token),
                                            _ptr(None if one_each or not paged else positions), *pages,
                                            _ptr(slots if paged else None), _ptr(kv_lens if paged else None), T, Hq,
                                            kv_heads, d, dv, page_size, *tail, _stream()), "attention_sigmoid_rowwise")


GATED_UMMA_TOKENS = 65  # prompts from this length on go to the tcgen05 kernel


def gated_ranks(seqs: int, kv_heads: int, group: int, max_kv_len: int, window: int, keep_first: int) -> int:
    """CTAs of a cluster that share a sequence's pages: as many as two CTAs per SM have room for at once, no CTA
    without a page. (At 32 sequences on 4 key heads, 1,088 keys: 27 us with 2 CTAs each, 39 with 3, whose clusters
    wait for one another; at 8 sequences 17 us with 8, 18 with 4, 23 with 2.)"""
    if force_gated_ranks is not None:
        return force_gated_ranks
    seen = min(max_kv_len, abs(window) + 63 + keep_first) if window else max_kv_len
    return max(1, min(8, -(-seen // 64), 2 * SM_COUNT // (seqs * kv_heads * -(-group // 16))))


def gated_decode_fused_supported(dtype, d: int, dv: int, kv, shaping: Shaping) -> bool:
    """True when the decode kernel can begin at the float32 projection: biases and a split-half rotation are
    all that stands between it and the attention."""
    return (not force_rowwise and not force_gated_split and dtype == torch.bfloat16 and kv is not None
            and shaping.taps is None and shaping.row_norm is None and shaping.head_weights is None
            and shaping.head_norm_eps is None and not shaping.adjacent_pairs
            and bool(library.load().lrm_attention_gated_supports(d, dv, kv.page_size)))


def gated(q, k, v, kv, kv_heads: int, dv: int, out, out_stride: int, form, gate, gate_stride: int, scale: float,
          window: int, out_scale: float, max_seq_len: int, max_kv_len: int, cu_seqlens, seq_of_token, positions, slots,
          kv_lens) -> None:
    """Softmax attention of an ops.SoftmaxForm (csrc/attention_gated.cu): packed keys k, v, or the cache view
    kv (one query per sequence where cu_seqlens is None). `out` and `gate` are pointers at first columns."""
    T, Hq, d = q.shape
    lib = library.load()
    paged = kv is not None
    one_each = paged and cu_seqlens is None
    keys, values = (kv.k, kv.v) if paged else (k, v)
    page_size = kv.page_size if paged else 64
    pages = (_ptr(kv.page_table), kv.page_table.shape[1], _ptr(slots), _ptr(kv_lens)) if paged else (None, 0, None, None)
    tail = (ctypes.c_float(scale), ctypes.c_float(form.cap or 0.0), window, form.keep_first, _ptr(form.sinks), gate,
            ctypes.c_longlong(gate_stride), int(form.gate_per_head), out, ctypes.c_longlong(out_stride),
            ctypes.c_float(out_scale))
    if (not force_rowwise and q.dtype == torch.bfloat16 and lib.lrm_attention_gated_supports(d, dv, page_size)
            and out_stride % 2 == 0 and all(t.data_ptr() % 16 == 0 for t in (q, keys, values)) and out.value % 4 == 0):
        ranks = 0
        if (not paged and not force_warp_level and max_seq_len >= GATED_UMMA_TOKENS and scale > 0 and out_stride % 8 == 0
                and out.value % 16 == 0 and lib.lrm_attention_gated_umma_supports(d, dv)):
            from . import gemm_dispatch
            gemm_dispatch.mark_status_dirty()
            _done(lib.lrm_attention_gated_umma(_ptr(q), _ptr(k), _ptr(v), _ptr(cu_seqlens), T, cu_seqlens.numel() - 1,
                                               max_seq_len, Hq, kv_heads, d, dv, *tail,
                                               _ptr(gemm_dispatch._status_word(q.device)), _stream()), "attention_gated_umma")
            return
        if one_each:
            ranks = gated_ranks(T, kv_heads, Hq // kv_heads, max_kv_len, window, form.keep_first)
        _done(lib.lrm_attention_gated(_ptr(q), _ptr(keys), _ptr(values), _ptr(None if one_each else cu_seqlens), *pages,
                                      T if one_each else cu_seqlens.numel() - 1, max_seq_len, Hq, kv_heads, d, dv, *tail,
                                      ranks, _stream()), "attention_gated_decode" if one_each else "attention_gated")
        return
    _done(lib.lrm_attention_gated_rowwise(_ptr(q), _ptr(keys), _ptr(values), _code(q.dtype), _ptr(cu_seqlens),
                                          _ptr(None if one_each else seq_of_token),
                                          _ptr(None if one_each or not paged else positions), *pages, T, Hq, kv_heads, d,
                                          dv, page_size, *tail, _stream()), "attention_gated_rowwise")


_cluster_room = {}


def _resident_clusters(head_dim: int, cluster: int, rows: int) -> int:
    """Clusters of this size, with `rows` query heads per kv head in a CTA, that the device holds
    at once (the region that partials are sent into grows with both); 0: cannot be launched."""
    key = (head_dim, cluster, rows)
    if key not in _cluster_room:
        _cluster_room[key] = int(library.load().lrm_attention_decode_cluster_resident(head_dim, cluster, rows))
    return _cluster_room[key]


def decode_fused_supported(dtype, head_dim: int, page_size: int, rotary: int, window) -> bool:
    """True when one cluster kernel can do rotation, cache write, attention and merge."""
    return (not force_rowwise and not force_unfused_decode and dtype == torch.bfloat16 and not window
            and bool(library.load().lrm_attention_decode_cluster_supports(head_dim, page_size, rotary)))


def decode_prefers_fused(seqs: int, kv_heads: int, group: int, head_dim: int, max_kv_len: int,
                         fill: int = 4) -> bool:
    """Whether the one-launch cluster kernel or the separate kernels are the faster way through a
    decode step's attention. A cluster has at most 16 CTAs, and a CTA keeps two pages in flight,
    which is worth 16-20 GB/s at head size 64 (25-30 at 128): a few sequences with a long context leave the
    cluster kernel with too few CTAs to draw the memory's bandwidth (measured: 112 CTAs 2.1 TB/s,
    224 CTAs 3.5, 320 CTAs 5.1, from 384 CTAs on 6.0-6.2), while the separate kernels cut a sequence
    into as many splits as fill the device and read at 6.6 TB/s (6.0 at head size 128), unless there are so many
    (sequence, head) pairs that each gets only two or three splits (256 pairs and more: 4.7-5.6).
    Against that stand their three launches: about 17 us before anything else counts, 8 us for the
    cluster kernel plus 0.35 us per page a CTA walks. Whole decode steps of the 1B shape, cluster
    kernel against separate kernels, ms: batch 1 at 16,000 keys 0.94 / 0.99, at 64,000 1.72 / 1.24;
    batch 4: 1.19 / 1.15 and 2.43 / 2.06; batch 8: 1.46 / 1.43 and 3.69 / 3.34; batch 32 at 16,000:
    3.85 / 4.50; batch 64: 6.92 / 7.29; at 4,000 keys the cluster kernel wins at every batch."""
    if force_cluster_size is not None:
        return True
    pages = max(1, -(-max_kv_len // 64))
    cluster = decode_cluster_size(seqs, kv_heads, group, head_dim, max_kv_len, fill)
    pairs = seqs * kv_heads * -(-group // 16)
    page_bytes = 4.0 * 64 * head_dim                       # a page of keys and one of values
    data = pairs * pages * page_bytes                      # bytes; rates below in bytes per us
    per_cta = 16e3 + 70.0 * head_dim                       # 20 GB/s at head size 64, 25 at 128
    fused = max(8.0 + 0.35 * -(-pages // cluster), data / min(6.1e6, pairs * cluster * per_cta))
    separate = max(17.0, data / (5.0e6 if pairs > 128 else 6.6e6 if head_dim <= 64 else 6.0e6) + 3.0)
    return fused <= separate


MAX_CLUSTER = 14  # clusters of 15 and 16 CTAs were measured slower as soon as a few hundred CTAs run


def decode_cluster_size(seqs: int, kv_heads: int, group: int, head_dim: int, max_kv_len: int, fill: int = 4) -> int:
    """CTAs per (sequence, kv head): any size up to MAX_CLUSTER (not only powers of two). Measured
    over batches of 1-32 and 600-8,000 keys, the kernel is fastest with about 400 CTAs in all at
    head size 64 (under 3 per SM, of the 4 that fit), about 500 when each walks many pages; more
    than fit at once cost a second round. `fill`: the sequences' mean length in quarters of the
    longest (4: about equal). Unequal sequences are handed out longest first, so the clusters that
    wait for room are those of the short sequences, and a size more pays: 16 sequences of 64-4,096
    keys, 1B shape: 1.20 ms per step with clusters of 4 against 1.25 with 3; 3B shape: 3.05-3.06 with
    5 or 4 against 3.16 with 3 (and 1.24-1.27 / 3.18 without the ordering, whatever the size)."""
    if force_cluster_size is not None:
        return force_cluster_size
    clusters = seqs * kv_heads * -(-group // 16)
    pages = max(1, -(-max_kv_len // 64))
    slots = (CTAS_PER_SM if head_dim <= 64 else 3) * SM_COUNT
    size = max(1, min(int(0.68 * slots / clusters + 0.5), pages, MAX_CLUSTER))
    if pages >= 16 * size:  # long rows of pages per CTA: bandwidth counts more than balance
        size = max(1, min(int(0.85 * slots / clusters + 0.5), pages, MAX_CLUSTER))
    while size > 1 and clusters > _resident_clusters(head_dim, size, min(group, 16)):
        size -= 1
    if fill < 4 and seqs > 1 and size < min(pages, MAX_CLUSTER):
        # as many more clusters may wait their turn as the short sequences leave room for
        if clusters * fill <= 4 * _resident_clusters(head_dim, size + 1, min(group, 16)):
            size += 1
    return size


def decode_fused(qkv, positions, inv_freq, rotary: int, kv, dest_rows, out, slots, kv_lens, max_kv_len: int,
                 q_heads: int, scale: float, order=None, fill: int = 4) -> None:
    B = qkv.shape[0]
    d = kv.head_dim
    cluster = decode_cluster_size(B, kv.kv_heads, q_heads // kv.kv_heads, d, max_kv_len, fill if order is not None else 4)
    _done(library.load().lrm_attention_decode_cluster(
        _ptr(qkv), _ptr(positions), _ptr(inv_freq), rotary, _ptr(kv.k), _ptr(kv.v), _ptr(dest_rows), _ptr(out),
        _ptr(kv.page_table), kv.page_table.shape[1], _ptr(slots), _ptr(kv_lens), B, q_heads, kv.kv_heads, d,
        kv.page_size, ctypes.c_float(scale), cluster, _ptr(order), _stream()), "attention_decode_cluster")


# --------------------------------------------------------------------------- one call for a mixer
def attend(projected, *, q_heads: int, kv_heads: int, head_dim: int, rotary, ctx, cache, writes_cache: bool,
           cache_entry: int, scale: float, window, projection=None, value_dim=None, bias=None, slopes=None,
           out_scale: float = 1.0, extras=None, values_are_keys: bool = False, shaping: Optional[Shaping] = None,
           chunk: Optional[int] = None, sigmoid_weights=None, form=None):
    """A layer's attention for one step: position rotation, cache write and attention, with the
    kernels chosen here for the step's phase, dtype and geometry. -> mixed heads [T, q_heads * d].

    projected: the step's fused [T, (q_heads + 2 kv_heads) * d] q|k|v projection when the layer
        writes its cache entry, else its [T, q_heads * d] queries (the entry was filled, in this
        step, by the layer that owns it).
    rotary: (inverse frequencies float32 [R/2], R) for a split-half rotation applied here, or None
        (no rotation: another scheme already transformed q and k, or there is none).
    ctx: the StepContext; cache: the KeyValueView of `cache_entry`; window: keys a query sees, or None.
    projection: (x, weight) instead of `projected` (then None) when nothing stands between the
        projection and the rotation: a prompt's product then rotates and stores in its epilogue.
    value_dim: head width of values when it is not head_dim; bias: float32 [projected width], added
        to the projection; slopes: float32 [q_heads], the linear distance penalty; out_scale: factor
        on the result; extras: per-head sinks and a query temperature (Extras); values_are_keys:
        the projection is q|k only and a key row is also its value row. With any of these the split
        kernel without rotation (csrc/qkv_store.cu) takes the place of the rotation kernel, and
        attention runs on the kernels that know them.
    shaping: a Shaping; the split kernel is then csrc/shaped_qkv.cu, which also rotates (`rotary`
        stays None) and takes the projection in float32. chunk: positions form chunks of this many,
        counted from position 0, and a query sees only the keys of its own chunk (`window` is then
        what the cache keeps, and the kernels are told the chunk as a negative window).
    sigmoid_weights: an ops.SigmoidWeights (with a `shaping`): no softmax, see there; the result may then
        go to columns of a tensor it names. form: an ops.SoftmaxForm (with a `shaping`), likewise.
    """
    from . import ops
    inv_freq, width = rotary if rotary is not None else (None, 0)
    phase = ctx.phase
    dv = head_dim if value_dim is None else value_dim
    if values_are_keys:
        dv = 0  # the projection has no value columns
    if chunk:
        window = -int(chunk)
    if (bias is not None or dv != head_dim or slopes is not None or out_scale != 1.0 or extras is not None
            or shaping is not None or chunk):
        if inv_freq is not None:
            from ..errors import UnsupportedError
            raise UnsupportedError("attention with a bias, a distance penalty or values of another width "
                                   "is built without rotation")
        if projection is not None:
            projected = ops.linear(*projection)
        prefill_phase = phase == "prefill"
        stored = dict(kv=cache if writes_cache else None,
                      dest_rows=ctx.dest_rows[cache.group] if writes_cache and cache is not None else None,
                      keep_packed=prefill_phase and writes_cache)
        if shaping is not None:
            s = shaping
            table = None
            in_one = (form is not None and phase == "decode" and writes_cache and projected.dtype == torch.float32
                      and gated_decode_fused_supported(ctx.runtime.dtype, head_dim, dv, cache, s))
            if s.inv_freq is not None:  # one table of angles per step and set of frequencies
                key = ("rope_table64", s.inv_freq.data_ptr(), s.magnitude)
                table = ctx.scratch.get(key)
                if table is None:
                    table = ctx.scratch[key] = ops.rope_table64(ctx.positions, s.inv_freq, s.magnitude)
            if in_one:  # biases, rotation, cache write and attention in one launch
                return ops.attention_gated_decode_fused(
                    projected, bias, table, s.rotary, q_heads, dv, form, cache, ctx.dest_rows[cache.group], ctx.slots,
                    ctx.kv_lens, ctx.max_kv_len, scale, window, out_scale)
            q, k, v = ops.shaped_qkv_store(
                projected, q_heads, kv_heads if writes_cache else 0, head_dim, dv, ctx.positions, ctx.runtime.dtype,
                bias=bias, taps=s.taps, tails=s.tails.state if s.tails is not None else None,
                cu_seqlens=ctx.cu_seqlens, seq_of_token=ctx.seq_of_token, slots=ctx.slots, row_norm=s.row_norm,
                row_eps=s.row_eps, head_weights=s.head_weights, head_weight_eps=s.head_weight_eps,
                inv_freq=s.inv_freq, rotary=s.rotary, adjacent_pairs=s.adjacent_pairs, head_norm_eps=s.head_norm_eps,
                table=table, magnitude=s.magnitude, **stored)
        else:
            q, k, v = ops.qkv_bias_store(projected, bias, q_heads, kv_heads if writes_cache else 0, head_dim, dv,
                                         **stored)
        if prefill_phase:
            if writes_cache:
                ctx.fresh_kv[cache_entry] = (k, k if values_are_keys else v)
            k, v = ctx.fresh_kv[cache_entry]
        if sigmoid_weights is not None or form is not None:
            where = dict(k=k, v=v) if prefill_phase else dict(kv=cache, slots=ctx.slots, kv_lens=ctx.kv_lens,
                                                              max_kv_len=ctx.max_kv_len)
            if phase != "decode":
                where.update(cu_seqlens=ctx.cu_seqlens, seq_of_token=ctx.seq_of_token, positions=ctx.positions)
            if form is not None:
                return ops.attention_gated(q, form, scale, window, out_scale, ctx.max_seq_len, **where)
            return ops.attention_sigmoid(q, sigmoid_weights, scale, window, out_scale, ctx.max_seq_len, **where)
        if prefill_phase:
            return ops.attention_prefill(q, k, v, ctx.cu_seqlens, ctx.seq_of_token, ctx.max_seq_len, scale, window,
                                         slopes, out_scale, extras)
        if phase == "decode":
            return ops.attention_decode(q, cache, ctx.slots, ctx.kv_lens, ctx.max_kv_len, scale, window, slopes,
                                        out_scale, extras)
        return ops.attention_extend(q, cache, ctx.cu_seqlens, ctx.seq_of_token, ctx.positions, ctx.slots,
                                    ctx.kv_lens, ctx.max_seq_len, scale, window, slopes, out_scale, extras)
    if projection is not None:
        x, weight = projection
        if (phase == "prefill" and writes_cache and x.dtype == torch.bfloat16 and weight.dtype == torch.bfloat16
                and width in (0, head_dim)):
            table = None
            if inv_freq is not None:   # one table of cosines and sines per step and rotation
                table = ctx.scratch.get(("rope_table", id(inv_freq)))
                if table is None:
                    table = ctx.scratch[("rope_table", id(inv_freq))] = ops.rope_table(ctx.positions, inv_freq)
            fused = ops.linear_rope_store(x, weight, q_heads, kv_heads, head_dim, table, cache,
                                          ctx.dest_rows[cache.group] if cache is not None else None)
            if fused is not None:
                q, k, v = fused
                ctx.fresh_kv[cache_entry] = (k, v)
                return ops.attention_prefill(q, k, v, ctx.cu_seqlens, ctx.seq_of_token, ctx.max_seq_len, scale, window)
        projected = ops.linear(x, weight)
    if writes_cache:
        if (phase == "decode" and cache is not None and projected.dtype == torch.bfloat16
                and decode_fused_supported(projected.dtype, head_dim, cache.page_size, width,
                                           window or cache.window)
                and decode_prefers_fused(projected.shape[0], kv_heads, q_heads // kv_heads, head_dim,
                                         ctx.max_kv_len, ctx.kv_fill)):
            # rotation, cache write, attention and the merge of the splits in one launch
            # the order comes with the step's arrays: the kernel reads it before it waits
            order = ctx.longest_first if projected.shape[0] > 1 else None
            return ops.attention_decode_fused(projected, q_heads, inv_freq, width, ctx.positions, cache,
                                              ctx.dest_rows[cache.group], ctx.slots, ctx.kv_lens,
                                              ctx.max_kv_len, scale, order, ctx.kv_fill)
        prefill = phase == "prefill"
        q, k, v = ops.rope_store(projected, q_heads, kv_heads, head_dim, inv_freq, width, ctx.positions,
                                 kv=cache, dest_rows=ctx.dest_rows[cache.group] if cache is not None else None,
                                 keep_packed=prefill)
        if prefill:
            ctx.fresh_kv[cache_entry] = (k, v)
    else:
        q, _, _ = ops.rope_store(projected, q_heads, 0, head_dim, inv_freq, width, ctx.positions,
                                 keep_packed=False)
        if phase == "prefill":
            k, v = ctx.fresh_kv[cache_entry]
    if phase == "prefill":
        return ops.attention_prefill(q, k, v, ctx.cu_seqlens, ctx.seq_of_token, ctx.max_seq_len, scale, window)
    if phase == "decode":
        return ops.attention_decode(q, cache, ctx.slots, ctx.kv_lens, ctx.max_kv_len, scale, window)
    return ops.attention_extend(q, cache, ctx.cu_seqlens, ctx.seq_of_token, ctx.positions, ctx.slots,
                                ctx.kv_lens, ctx.max_seq_len, scale, window)
