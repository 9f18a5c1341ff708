"""Every mechanism of the Munupel decoder alone on the GPU, with inputs made so that a fault shows."""
import numpy as np
import pytest
import torch

import helpers
import plain_munupel as P

pytestmark = pytest.mark.gpu
DEV = "cuda"
F64 = torch.float64
F32, BF16 = torch.float32, torch.bfloat16


def i32(*values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def worst(got, want):
    got, want = got.detach().cpu().double(), want.double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    return float((got - want).abs().max() / want.abs().max().clamp(min=1e-30))


def visibility(span, keep):
    """sees(i) of the plain implementation for a window (> 0), a chunk (< 0) or neither."""
    if span is None:
        return lambda i: P.chunk_sees(i, None)
    return (lambda i: P.chunk_sees(i, -span)) if span < 0 else (lambda i: P.window_sees(i, span, keep))


def fast_attention(q, k, v, scale, span, keep, cap, sinks):
    """The plain attention, all queries of a head at once (the same mask, row by row)."""
    T, H, _ = q.shape
    mask = torch.zeros(T, T, dtype=torch.bool)
    for i in range(T):
        mask[i, visibility(span, keep)(i)] = True
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // k.shape[1])
        s = P.softcap((q[:, h] @ k[:, g].T) * scale, cap).masked_fill(~mask, -torch.inf)
        if sinks is not None:
            s = torch.cat([s, sinks[h].expand(T, 1)], dim=1)
        out[:, h] = torch.softmax(s, dim=1)[:, :T] @ v[:, g]
    return out


def test_the_whole_row_form_of_the_plain_attention_is_the_plain_attention():
    gen = torch.Generator().manual_seed(1)
    rand = lambda *s: torch.randn(*s, generator=gen, dtype=F64)  # noqa: E731
    q, k, v, sinks = rand(30, 4, 6), rand(30, 2, 6), rand(30, 2, 5), rand(4)
    for span, keep, cap, snk in ((5, 3, None, sinks), (-7, 0, 2.0, None), (None, 0, 1.0, sinks)):
        assert torch.allclose(fast_attention(q, k, v, 0.7, span, keep, cap, snk), P.attention(q, k, v, 0.7, visibility(span, keep), cap, snk))


class Ways:
    """One attention problem run as a prompt, as portions, and as decode steps, over keys stored in a cache whose
    other rows and pages hold values that must not be seen."""

    def __init__(self, dtype, q, k, v, form, scale, span, keep, out_scale):
        from llama_rs_metal_b200.cache import Cache
        from llama_rs_metal_b200.parts.base import KeyValueRequest
        self.dtype, self.q, self.k, self.v = dtype, q, k, v
        self.form, self.scale, self.span, self.out_scale = form, scale, span, out_scale
        (L, self.H, d), (_, self.G, dv) = q.shape, v.shape
        self.L, self.d, self.dv = L, d, dv
        window = None if span is None else abs(span)
        self.cache = Cache([KeyValueRequest(self.G, d, window, None if dv == d else dv, keep_first=keep)], dtype, torch.device(DEV),
                           512, 3, 512)
        for t in [*self.cache.kv_groups[0].k.values(), *self.cache.kv_groups[0].v.values()]:
            t.fill_(float("nan"))                              # rows nobody stored must not reach a product
        self.cache.open_slot()
        self.slot = self.cache.open_slot()

    def prompt(self):
        from llama_rs_metal_b200.kernels import ops
        cu, seq_of = i32(0, self.L), torch.zeros(self.L, dtype=torch.int32, device=DEV)
        return ops.attention_gated(self.q, self.form(0, self.L), self.scale, self.span, self.out_scale, self.L, k=self.k, v=self.v,
                                   cu_seqlens=cu, seq_of_token=seq_of).reshape(self.L, self.H, self.dv)

    def store(self, at, n):
        from llama_rs_metal_b200.kernels import ops
        dest = torch.tensor(self.cache.destination_rows([self.slot], [at], [n])[0], device=DEV)
        packed = torch.cat([x[at:at + n].reshape(n, -1) for x in (self.q, self.k, self.v)], dim=1).contiguous()
        out, _, _ = ops.qkv_bias_store(packed, None, self.H, self.G, self.d, self.dv, kv=self.cache.view(0), dest_rows=dest,
                                       keep_packed=False)
        self.cache.commit([(self.slot, at + n)])
        return out

    def cached(self, first, stop, portion):
        """Tokens first .. stop - 1 in portions (1: decode steps) behind a prompt of `first` tokens."""
        from llama_rs_metal_b200.kernels import ops
        cache, slot, rows = self.cache, self.slot, []
        cache.reset_slot(slot)
        if first:
            cache.grow([(slot, first)])
            cache.sync()
            self.store(0, first)
        for at in range(first, stop, portion):
            n = min(portion, stop - at)
            cache.grow([(slot, at + n, at)])
            cache.sync()
            q = self.store(at, n)
            where = dict(kv=cache.view(0), slots=i32(slot), kv_lens=i32(at + n), max_kv_len=512)
            if portion > 1:
                where.update(cu_seqlens=i32(0, n), seq_of_token=torch.zeros(n, dtype=torch.int32, device=DEV),
                             positions=torch.arange(at, at + n, dtype=torch.int32, device=DEV))
            rows.append(ops.attention_gated(q, self.form(at, n), self.scale, self.span, self.out_scale, n, **where)
                        .reshape(n, self.H, self.dv))
        return torch.cat(rows)


# (dtype, H, G, d, dv, span (window > 0, chunk < 0), kept keys, cap, sinks, gate)
CASES = [
    (F32, 4, 2, 24, 40, 7, 3, 4.0, True, "element"), (F32, 3, 1, 96, 64, -64, 0, None, False, "head"), (F32, 2, 2, 160, 200, 70, 65, 9.0, True, None),
    (F32, 2, 1, 16, 8, None, 0, 3.0, True, "head"), (BF16, 4, 2, 64, 64, 70, 5, None, True, "head"), (BF16, 4, 4, 32, 32, -64, 0, 8.0, False, "element"),
    (BF16, 2, 1, 128, 128, 100, 64, 20.0, True, "element"), (BF16, 3, 3, 96, 32, 65, 130, None, True, "head"),
    (BF16, 20, 1, 40, 56, -70, 0, 5.0, False, "element"), (BF16, 4, 2, 24, 128, 1, 1, None, True, "head"), (BF16, 2, 1, 128, 8, -1, 0, 6.0, False, "element"),
    (BF16, 4, 2, 96, 96, None, 0, 12.0, False, None), (BF16, 4, 2, 20, 30, 64, 10, 7.0, True, "element"), (BF16, 34, 2, 64, 96, -96, 0, None, True, "head"),
    (BF16, 4, 1, 56, 72, 128, 63, None, False, "head"), (BF16, 2, 2, 160, 136, 40, 20, 4.0, True, "element"),
]


@pytest.mark.parametrize("dtype,H,G,d,dv,span,keep,cap,sink,gate", CASES)
def test_a_key_that_stands_out_on_both_sides_of_every_edge(dtype, H, G, d, dv, span, keep, cap, sink, gate):
    """Keys that stand out, one at a time: the last kept one and the first that is not, one in the middle of a
    page, the last and the first of a page. Each scores far above the others and has a value of its own, so that
    it makes most of every output that sees it. Prompts on every kernel, portions of two and seven, decode steps
    on every number of CTAs, all around the query where the key leaves the window or its chunk ends."""
    from llama_rs_metal_b200.kernels import attention_dispatch, ops
    L, gap, out_scale = 330, 3, 0.7
    gen = torch.Generator().manual_seed(d + 3 * dv + H)
    rand = lambda *s: torch.randn(*s, generator=gen, dtype=F64)  # noqa: E731
    r = lambda t: t.to(dtype).to(DEV).contiguous()  # noqa: E731
    tol = 2e-5 if dtype == F32 else 2e-2
    tiled = dtype == BF16 and d % 8 == 0 and dv % 8 == 0 and max(d, dv) <= 128
    width = H if gate == "head" else H * dv
    size = abs(span) if span else 200
    spikes = sorted({s for s in (keep - 1, keep, 3, 127, 128, 150) if s >= 0})
    for spike in spikes:
        if span is None or span > 0:
            edge = spike + size                                # the first query that does not see it (unless it is kept)
        else:
            edge = (spike // size + 1) * size
        first, stop = min(max(edge - 3, 1), L - 8), min(max(edge - 3, 1), L - 8) + 8
        q, k, v = rand(L, H, d) * 0.2, rand(L, G, d) * 0.2, rand(L, G, dv)
        q[:, :, -1] = 3.0                                      # (behind any rotation)
        k[:, :, -1] = -1.0
        k[spike, :, -1] = 2.5
        v[spike] *= 4.0
        gates, sinks = rand(L, gap + width), rand(H) + 1.0
        rq, rk, rv, rg, rs = r(q), r(k), r(v), gates.float().to(DEV).contiguous(), sinks.float().to(DEV)
        ref = fast_attention(*(x.cpu().double() for x in (rq, rk, rv)), 1.0, span, keep, cap, rs.cpu().double() if sink else None) * out_scale
        if gate:
            factor = torch.sigmoid(rg.cpu().double()[:, gap:])
            ref = ref * (factor[:, :, None] if gate == "head" else factor.reshape(L, H, dv))

        def form(at, n, out=None):
            columns = (rg[at:at + n].contiguous(), gap) if gate else None
            return ops.SoftmaxForm(cap, rs if sink else None, keep, columns, gate == "head", (out, gap + 1) if out is not None else None)
        ways = Ways(dtype, rq, rk, rv, form, 1.0, span, keep, out_scale)
        for warp_level in ((False, True) if tiled else (False,)):
            attention_dispatch.force_warp_level = warp_level
            try:
                assert worst(ways.prompt(), ref) <= tol, f"prompt, key {spike}, warp level {warp_level}"
            finally:
                attention_dispatch.force_warp_level = False
        pad = -(gap + 1 + H * dv) % 8                           # rows of whole 16-byte pieces, and rows that are not
        for wide in (torch.full((L, gap + 1 + H * dv + pad), 5.0, dtype=dtype, device=DEV),
                     torch.full((L, gap + 1 + H * dv + pad + 1), 5.0, dtype=dtype, device=DEV)):
            ops.attention_gated(rq, form(0, L, wide), 1.0, span, out_scale, L, k=rk, v=rv, cu_seqlens=i32(0, L),
                                seq_of_token=torch.zeros(L, dtype=torch.int32, device=DEV))
            columns = slice(gap + 1, gap + 1 + H * dv)
            assert worst(wide[:, columns].reshape(L, H, dv), ref) <= tol
            wide[:, columns] = 5.0
            assert float((wide - 5.0).abs().max()) == 0.0, "columns of someone else were written"
        for portion, ranks in ((1, None), (1, 1), (1, 3), (1, 8), (2, None), (7, None)):
            if ranks is not None and not tiled:
                continue
            attention_dispatch.force_gated_ranks = ranks
            try:
                got = ways.cached(first, stop, portion)
                assert worst(got, ref[first:stop]) <= tol, f"portions of {portion} on {ranks} CTAs, key {spike}"
            finally:
                attention_dispatch.force_gated_ranks = None


@pytest.mark.parametrize("dtype,d,dv,span,keep", [(F32, 24, 16, 50, 9), (BF16, 64, 32, 50, 9), (BF16, 128, 96, -40, 0), (BF16, 40, 128, 64, 64), (BF16, 12, 20, 30, 2)])
def test_packed_prompts_do_not_see_one_another(dtype, d, dv, span, keep):
    from llama_rs_metal_b200.kernels import attention_dispatch, ops
    lengths, H, G = [70, 1, 200, 64, 129], 4, 2
    gen = torch.Generator().manual_seed(d)
    r = lambda *s: torch.randn(*s, generator=gen).to(dtype)  # noqa: E731
    T = sum(lengths)
    q, k, v, sinks = r(T, H, d), r(T, G, d), r(T, G, dv), torch.randn(H, generator=gen)
    cu = [0]
    for n in lengths:
        cu.append(cu[-1] + n)
    seq_of = torch.repeat_interleave(torch.arange(5, dtype=torch.int32), torch.tensor(lengths)).to(DEV)
    want = torch.cat([fast_attention(q[a:b].double(), k[a:b].double(), v[a:b].double(), 0.4, span, keep, 3.0, sinks.double())
                      for a, b in zip(cu, cu[1:])])
    for warp_level in (False, True):
        attention_dispatch.force_warp_level = warp_level
        try:
            got = ops.attention_gated(q.to(DEV), ops.SoftmaxForm(3.0, sinks.to(DEV), keep), 0.4, span, 1.0, max(lengths), k=k.to(DEV),
                                      v=v.to(DEV), cu_seqlens=i32(*cu), seq_of_token=seq_of)
        finally:
            attention_dispatch.force_warp_level = False
        assert worst(got.reshape(T, H, dv), want) < (1e-5 if dtype == F32 else 2e-2)


def test_a_maximum_that_moves_far_from_tile_to_tile():
    """Scores that climb by dozens from one tile of keys to the next, and scores that fall: every rescaling of what
    was added up before; sinks above and below all of them."""
    from llama_rs_metal_b200.kernels import attention_dispatch, ops
    L, H, d = 300, 4, 64
    gen = torch.Generator().manual_seed(9)
    q, k, v = (torch.randn(L, H, d, generator=gen).to(BF16) * 0.1 for _ in range(3))
    v = (v * 10).to(BF16)
    q[:, :, 0] = 4.0
    steps = torch.arange(L) // 64
    k[:, 0, 0], k[:, 1, 0], k[:, 2, 0] = 10.0 * steps, -10.0 * steps, 20.0 * (steps % 2)
    sinks = torch.tensor([120.0, -3.0, -200.0, 1.0])
    ref = fast_attention(q.double(), k.double(), v.double(), 1.0, None, 0, None, sinks.double())
    for warp_level in (False, True):
        attention_dispatch.force_warp_level = warp_level
        try:
            got = ops.attention_gated(q.to(DEV), ops.SoftmaxForm(sinks=sinks.to(DEV)), 1.0, None, 1.0, L, k=k.to(DEV), v=v.to(DEV),
                                      cu_seqlens=i32(0, L), seq_of_token=torch.zeros(L, dtype=torch.int32, device=DEV))
        finally:
            attention_dispatch.force_warp_level = False
        assert worst(got.reshape(L, H, d), ref) < 2e-2


# --------------------------------------------------------------------------- the split with a rotation's magnitude
@pytest.mark.parametrize("dtype,Hq,Hk,d,dv,rotary,gap", [(F32, 3, 1, 10, 6, 6, 1), (F32, 4, 2, 16, 8, 8, 4), (BF16, 4, 2, 64, 32, 48, 4), (BF16, 6, 3, 40, 56, 24, 0),
                                                         (BF16, 2, 2, 96, 96, 20, 3), (BF16, 5, 1, 128, 64, 0, 8)])
@pytest.mark.parametrize("with_table", [True, False])
def test_split_with_biases_and_a_scaled_rotation(dtype, Hq, Hk, d, dv, rotary, gap, with_table):
    """Biases, a rotation of part of every query and key head whose cosines and sines have a magnitude, the split,
    and the rows of the cache, from a projection with further columns behind the row."""
    from llama_rs_metal_b200.cache import Cache
    from llama_rs_metal_b200.kernels import ops
    from llama_rs_metal_b200.parts.base import KeyValueRequest
    T, at = 150, 70
    gen = torch.Generator().manual_seed(d + rotary)
    width = Hq * d + Hk * (d + dv)
    proj, bias = torch.randn(T, width + gap, generator=gen), torch.randn(width, generator=gen)
    rot = helpers._scaled_rotation(rotary, 300.0, (4.0, 128, 8.0, 1.0)) if rotary else None
    pos = torch.arange(at, at + T)
    row = (proj[:, :width] + bias).double()
    q, k, v = row[:, :Hq * d].reshape(T, Hq, d), row[:, Hq * d:Hq * d + Hk * d].reshape(T, Hk, d), row[:, -Hk * dv:].reshape(T, Hk, dv)
    args = {}
    if rot:
        q, k = P.rotate_halves(q, pos, rot), P.rotate_halves(k, pos, rot)
        freqs, magnitude = P.rotation(rot)
        args = dict(inv_freq=torch.tensor(freqs, dtype=F64, device=DEV), rotary=rotary, magnitude=magnitude)
        if with_table:
            args["table"] = ops.rope_table64(pos.int().to(DEV), args["inv_freq"], magnitude)
    cache = Cache([KeyValueRequest(Hk, d, None, None if d == dv else dv)], dtype, torch.device(DEV), 512, 1, 512)
    slot = cache.open_slot()
    cache.grow([(slot, at + T)])
    dest = torch.tensor(cache.destination_rows([slot], [at], [T])[0], device=DEV)
    got = ops.shaped_qkv_store(proj.to(DEV), Hq, Hk, d, dv, pos.int().to(DEV), dtype, bias=bias.to(DEV), kv=cache.view(0), dest_rows=dest, **args)
    cache.commit([(slot, at + T)])
    tol = 1e-5 if dtype == F32 else 6e-3
    for name, g, w in zip("qkv", got, (q, k, v)):
        assert worst(g, w) <= tol, name
    kept_k, kept_v = cache.snapshot(slot, 0)
    assert torch.equal(kept_k[at:], got[1].float().cpu()) and torch.equal(kept_v[at:], got[2].float().cpu())


@pytest.mark.parametrize("H,G,d,dv,rotary,span,keep,cap,sink,gate", [
    (4, 2, 64, 32, 24, 70, 5, None, True, "head"), (20, 1, 40, 56, 40, -64, 0, 5.0, False, "element"), (36, 2, 128, 128, 0, 100, 64, None, True, "head"),
    (3, 3, 96, 96, 96, -130, 0, 9.0, False, "element"), (2, 1, 8, 16, 2, 1, 0, None, True, "head"), (4, 4, 32, 64, 32, None, 0, 3.0, False, None)])
def test_decode_steps_that_begin_at_the_projection(H, G, d, dv, rotary, span, keep, cap, sink, gate):
    """The one-launch decode step against the split and the attention in launches of their own: the same rows in the
    cache bit for bit, the same outputs to rounding, for unequal sequences across page borders and freed pages."""
    from llama_rs_metal_b200.cache import Cache
    from llama_rs_metal_b200.kernels import attention_dispatch, ops
    from llama_rs_metal_b200.parts.base import KeyValueRequest
    lengths, width, gcols = [1, 63, 64, 190], H * d + G * (d + dv), H * dv if gate == "element" else H if gate else 0
    B, stride = len(lengths), width + gcols + (-(width + gcols)) % 32
    gen = torch.Generator().manual_seed(H + d)
    bias = torch.randn(width, generator=gen).to(DEV) if cap else None
    sinks = torch.randn(H, generator=gen).to(DEV) if sink else None
    inv = (50.0 ** (-torch.arange(rotary // 2, dtype=F64) * 2 / max(rotary, 1))).to(DEV)
    window = None if span is None else abs(span)
    caches = [Cache([KeyValueRequest(G, d, window, None if dv == d else dv, keep_first=keep)], BF16, torch.device(DEV), 1024, 5, 512) for _ in range(2)]
    for cache in caches:
        for t in [*cache.kv_groups[0].k.values(), *cache.kv_groups[0].v.values()]:
            t.fill_(float("nan"))
        slots = [cache.open_slot() for _ in range(5)][1:]
        filler = torch.Generator().manual_seed(3)
        for slot, n in zip(slots, lengths):
            cache.grow([(slot, n)])
            dest = torch.tensor(cache.destination_rows([slot], [0], [n])[0], device=DEV)
            rows = torch.randn(n, width, generator=filler).to(BF16).to(DEV)
            ops.qkv_bias_store(rows, None, H, G, d, dv, kv=cache.view(0), dest_rows=dest, keep_packed=False)
            cache.commit([(slot, n)])
    at = list(lengths)
    for step in range(5):
        proj = torch.randn(B, stride, generator=gen).to(DEV)
        pos = i32(*at)
        table = ops.rope_table64(pos, inv, 1.2) if rotary else None
        form = ops.SoftmaxForm(cap, sinks, keep, (proj, width) if gate else None, gate == "head")
        outs = []
        for fused, cache in zip((True, False), caches):
            before, rows = cache.grow_by_one(np.array(slots))
            cache.sync()
            dest, lens = torch.tensor(rows[0], device=DEV), i32(*[n + 1 for n in at])
            where = dict(kv=cache.view(0), slots=i32(*slots), kv_lens=lens, max_kv_len=512)
            if fused:
                attention_dispatch.force_gated_ranks = (None, 1, 2, 5, 8)[step]
                outs.append(ops.attention_gated_decode_fused(proj, bias, table, rotary, H, dv, form, cache.view(0), dest, where["slots"],
                                                             lens, 512, 0.2, span, 0.8))
                attention_dispatch.force_gated_ranks = None
            else:
                q, _, _ = ops.shaped_qkv_store(proj, H, G, d, dv, pos, BF16, bias=bias, inv_freq=inv if rotary else None, rotary=rotary,
                                               table=table, magnitude=1.2, kv=cache.view(0), dest_rows=dest, keep_packed=False)
                outs.append(ops.attention_gated(q, form, 0.2, span, 0.8, 1, **where))
            cache.commit_lengths(np.array(slots), before + 1)
        assert worst(outs[0], outs[1].cpu()) < 1e-2, f"step {step}"
        at = [n + 1 for n in at]
    for slot in slots:
        for a, b in zip(caches[0].snapshot(slot, 0), caches[1].snapshot(slot, 0)):
            assert torch.equal(torch.nan_to_num(a), torch.nan_to_num(b))


# --------------------------------------------------------------------------- joined products and the moving norm
@pytest.mark.parametrize("M", [1, 5, 8, 13, 16, 33, 64, 70, 300, 1100])
@pytest.mark.parametrize("K,plain,ff,extra", [(72, 100, 40, 8), (192, 352, 448, 64), (1024, 1000, 2048, 512)])
def test_one_product_for_a_projection_and_a_gate(M, K, plain, ff, extra):
    from llama_rs_metal_b200.kernels import gemm_dispatch, ops
    from llama_rs_metal_b200.parts.linear import SplitLinear
    gen = torch.Generator().manual_seed(M + K)
    x = torch.randn(M, K, generator=gen).to(BF16)
    w, g, u = (torch.randn(n, K, generator=gen).to(BF16) * K ** -0.5 for n in (plain, ff, ff))
    fused = torch.stack([g.reshape(ff // 8, 8, K), u.reshape(ff // 8, 8, K)], dim=1).reshape(2 * ff, K)
    both = SplitLinear(w.to(DEV), fused.to(DEV))
    want = x.double() @ w.double().T
    gate = x.double() @ g.double().T
    inner = gate * torch.sigmoid(gate) * (x.double() @ u.double().T)
    for tiled in (False, True):
        gemm_dispatch.force_tiled = tiled
        try:
            row = torch.full((M, ff + extra), 3.0, dtype=BF16, device=DEV)
            got = both(x.to(DEV), row)
            gemm_dispatch.check_status()
        finally:
            gemm_dispatch.force_tiled = False
        assert got.dtype == F32 and worst(got[:, :plain], want) < 1e-5 and not got[:, plain:].any()
        assert worst(row[:, :ff], inner) < 6e-3 and float((row[:, ff:] - 3.0).abs().max()) == 0.0


@pytest.mark.parametrize("tile", [128, 192, 256, 512, "pair"])
def test_every_tile_of_the_tensor_core_products_divides_at_the_split(tile):
    from llama_rs_metal_b200.kernels import gemm_dispatch, ops
    M, K, plain, ff = 520, 256, 352, 480
    gen = torch.Generator().manual_seed(5)
    x = torch.randn(M, K, generator=gen).to(BF16).to(DEV)
    w = (torch.randn(plain + 2 * ff, K, generator=gen) / 16).to(BF16).to(DEV)
    if tile == "pair" and gemm_dispatch.pair_room() == 0:
        pytest.skip("no pairs of SMs")
    want_row = torch.empty((M, ff + 16), dtype=BF16, device=DEV)
    want = ops.linear_split(x, w, plain, want_row)
    gemm_dispatch.umma_width = tile
    try:
        row = torch.empty_like(want_row)
        got = ops.linear_split(x, w, plain, row)
        gemm_dispatch.check_status()
    finally:
        gemm_dispatch.umma_width = None
    assert worst(got, want.cpu()) < 1e-5 and worst(row[:, :ff], want_row[:, :ff].cpu()) < 6e-3
    assert worst(got, (x.cpu().double() @ w[:plain].cpu().double().T)) < 1e-5


@pytest.mark.parametrize("hidden", [72, 256, 1000, 2048, 4096, 9000])
@pytest.mark.parametrize("slices", [0, 1, 3])
def test_a_norm_that_moves_the_stream_on(hidden, slices):
    """The row is normalized without the vector that is added to the stream behind it, the slices of a product are
    added first, and the updated stream is written back."""
    from llama_rs_metal_b200.kernels import ops
    gen = torch.Generator().manual_seed(hidden)
    x, w, b, add = torch.randn(9, hidden, generator=gen) * 3 + 1, *(torch.randn(hidden, generator=gen) for _ in range(3))
    parts = torch.randn(slices, 9, hidden, generator=gen) if slices else None
    stream = x.double() + (parts.double().sum(0) if slices else 0.0)
    want = P.layer_norm(stream, w.double(), b.double(), 1e-5)
    for dtype in (F32, BF16):
        moved = x.to(DEV)
        y = ops.layer_norm(moved, w.to(DEV), b.to(DEV), 1e-5, dtype, partials=parts.to(DEV) if slices else None, add=add.to(DEV))
        assert worst(y, want) < (2e-6 if dtype == F32 else 5e-3)
        assert worst(moved, stream + add.double()) < 1e-6
