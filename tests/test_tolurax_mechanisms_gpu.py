"""Every mechanism of the Tolurax decoder alone on the GPU, with inputs made so that a fault shows."""
import pytest
import torch

import plain_tolurax as P

pytestmark = pytest.mark.gpu
DEV = "cuda"
F64 = torch.float64


def i32(*values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def worst(got, want):
    got, want = got.detach().cpu().double(), want.double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    return float((got - want).abs().max() / want.abs().max().clamp(min=1e-30))


# --------------------------------------------------------------------------- sigmoid attention
def plain_attention(q, k, v, scale, offset, window, gate, out_scale):
    L, H, _ = q.shape
    out = P.sigmoid_attention(q, k, v, scale, offset, window).reshape(L, H, -1)
    return out * torch.sigmoid(gate.reshape(out.shape)) * out_scale


@pytest.mark.parametrize("dtype,H,G,d,dv,window", [
    (torch.float32, 4, 2, 24, 40, 7), (torch.float32, 3, 1, 96, 96, 64), (torch.float32, 2, 2, 16, 8, 70),
    (torch.bfloat16, 4, 2, 64, 64, 70), (torch.bfloat16, 4, 4, 32, 32, 64), (torch.bfloat16, 2, 1, 128, 128, 100),
    (torch.bfloat16, 3, 3, 96, 96, 65), (torch.bfloat16, 20, 1, 64, 64, 40), (torch.bfloat16, 4, 2, 48, 16, 65),
    (torch.bfloat16, 2, 1, 64, 64, 1), (torch.bfloat16, 4, 2, 96, 96, None), (torch.float32, 2, 1, 160, 200, None)])
def test_a_key_that_stands_out_just_inside_and_just_outside_a_window(dtype, H, G, d, dv, window):
    """One key scores so high, and its value is so large, that it makes most of every output that sees it, and
    the other keys score far below zero; with a window it is seen at distance window - 1 and no longer at
    window. Prompts, decoding (every number of CTAs per sequence) and portions of three, with the edges on
    and next to page borders; gate and factor applied, results in columns of a wider tensor."""
    from llama_rs_metal_b200.cache import Cache
    from llama_rs_metal_b200.kernels import attention_dispatch, ops
    from llama_rs_metal_b200.parts.base import KeyValueRequest
    L, gap = 330, 5
    gen = torch.Generator().manual_seed(d + dv + H)
    rand = lambda *s: torch.randn(*s, generator=gen, dtype=F64)  # noqa: E731
    span = window or 200
    for spike in (128 - span + 64 if span < 190 else 3, 127):
        edge = spike + span                                   # the first query that does not see the key
        if edge + 6 >= L:
            continue
        q, k, v = rand(L, H, d) * 0.2, rand(L, G, d) * 0.2, rand(L, G, dv) * 0.3
        q[:, :, 0], k[:, :, 0] = 3.0, -1.0                    # scores near -3: small weights
        k[spike, :, 0] = 3.0                                  # score near 9: weight 1
        v[spike] = 9.0
        offset, gate = rand(H), rand(L, gap + H * dv)
        r = lambda t: t.to(dtype).to(DEV).contiguous()  # noqa: E731
        rq, rk, rv = r(q), r(k), r(v)
        rgate, roffset = gate.float().to(DEV).contiguous(), offset.float().to(DEV)
        ref = plain_attention(rq.cpu().double(), rk.cpu().double(), rv.cpu().double(), 1.0, roffset.cpu().double(), window,
                              rgate.cpu().double()[:, gap:], 0.7)
        share = torch.sigmoid(rgate.cpu().double()[:, gap:]).reshape(L, H, dv) * 0.7
        if window:
            assert float((ref[edge - 1] / share[edge - 1]).min()) > 6.0 and float((ref[edge] / share[edge]).abs().max()) < 6.0
        tol = 2e-5 if dtype == torch.float32 else 2e-2
        if dtype == torch.bfloat16 and window is None:
            tol = 3e-2                                        # hundreds of small weights, each rounded

        def weights(at, n, out=None):
            return ops.SigmoidWeights(roffset, (rgate[at:at + n].contiguous(), gap), (out, gap + 1) if out is not None else None)
        cu, seq_of = i32(0, L), torch.zeros(L, dtype=torch.int32, device=DEV)
        got = ops.attention_sigmoid(rq, weights(0, L), 1.0, window, 0.7, L, k=rk, v=rv, cu_seqlens=cu, seq_of_token=seq_of)
        assert worst(got.reshape(L, H, dv), ref) <= tol, f"prompt, key {spike}"
        wide = torch.full((L, gap + 1 + H * dv + 2), 5.0, dtype=dtype, device=DEV)
        ops.attention_sigmoid(rq, weights(0, L, wide), 1.0, window, 0.7, L, k=rk, v=rv, cu_seqlens=cu, seq_of_token=seq_of)
        assert worst(wide[:, gap + 1:-2].reshape(L, H, dv), ref) <= tol
        assert float((wide[:, :gap + 1] - 5.0).abs().max()) == 0.0 and float((wide[:, -2:] - 5.0).abs().max()) == 0.0
        cache = Cache([KeyValueRequest(G, d, window, None if dv == d else dv)], dtype, torch.device(DEV), 512, 2, 512)
        cache.open_slot()
        slot = cache.open_slot()

        def store(at, n):
            dest = torch.tensor(cache.destination_rows([slot], [at], [n])[0], device=DEV)
            packed = torch.cat([x[at:at + n].reshape(n, -1) for x in (rq, rk, rv)], dim=1).contiguous()
            out, _, _ = ops.qkv_bias_store(packed, None, H, G, d, dv, kv=cache.view(0), dest_rows=dest, keep_packed=False)
            cache.commit([(slot, at + n)])
            return out
        for portion, ranks in ((1, None), (1, 1), (1, 3), (1, 8), (3, None)):
            if ranks is not None and (dtype == torch.float32 or dv != d or d == 48):
                continue
            attention_dispatch.force_sigmoid_ranks = ranks
            try:
                cache.reset_slot(slot)
                first, rows = edge - 4, []
                cache.grow([(slot, first)])
                cache.sync()
                store(0, first)
                for at in range(first, first + 9, portion):
                    n = portion
                    cache.grow([(slot, at + n, at)])
                    cache.sync()
                    qn = store(at, n)
                    where = dict(kv=cache.view(0), slots=i32(slot), kv_lens=i32(at + n), max_kv_len=512)
                    if portion > 1:
                        where.update(cu_seqlens=i32(0, n), seq_of_token=torch.zeros(n, dtype=torch.int32, device=DEV),
                                     positions=torch.arange(at, at + n, dtype=torch.int32, device=DEV))
                    rows.append(ops.attention_sigmoid(qn, weights(at, n), 1.0, window, 0.7, n, **where).reshape(n, H, dv))
                assert worst(torch.cat(rows), ref[first:first + 9]) <= tol, f"portions of {portion} on {ranks} CTAs, key {spike}"
            finally:
                attention_dispatch.force_sigmoid_ranks = None


@pytest.mark.parametrize("dtype,d", [(torch.float32, 24), (torch.bfloat16, 64), (torch.bfloat16, 128), (torch.bfloat16, 96)])
def test_packed_prompts_do_not_see_one_another(dtype, d):
    from llama_rs_metal_b200.kernels import ops
    lengths, H, G = [70, 1, 130, 64], 4, 2
    gen = torch.Generator().manual_seed(d)
    r = lambda *s: torch.randn(*s, generator=gen).to(dtype)  # noqa: E731
    T = sum(lengths)
    q, k, v = r(T, H, d) * 0.5, r(T, G, d), r(T, G, d)
    offset = torch.randn(H, generator=gen)
    cu = [0]
    for n in lengths:
        cu.append(cu[-1] + n)
    seq_of = torch.repeat_interleave(torch.arange(4, dtype=torch.int32), torch.tensor(lengths)).to(DEV)
    got = ops.attention_sigmoid(q.to(DEV), ops.SigmoidWeights(offset.to(DEV)), 0.3, 50, 1.0, max(lengths), k=k.to(DEV),
                                v=v.to(DEV), cu_seqlens=i32(*cu), seq_of_token=seq_of)
    want = torch.cat([P.sigmoid_attention(q[a:b].double(), k[a:b].double(), v[a:b].double(), 0.3, offset.double(), 50)
                      for a, b in zip(cu, cu[1:])])
    assert worst(got, want) < (1e-5 if dtype == torch.float32 else 2e-2)


# --------------------------------------------------------------------------- the two recurrences
def carried(parts, run, lengths, heads_state, slot_of):
    """Run a scan over two sequences (with a sequence of padding between them) in steps of the given lengths;
    -> outputs per sequence, and the state storage."""
    state = torch.full((5, *heads_state), 7.0, dtype=torch.float32, device=DEV)
    state[slot_of] = 0.0
    slots = i32(slot_of[0], -1, slot_of[1])
    at, outs, pad = 0, [[], []], 4
    for n in lengths:
        step = {}
        for name, (a, b) in parts.items():
            filler = torch.ones((pad, *a.shape[1:]), dtype=F64)
            step[name] = torch.cat([a[at:at + n], filler, b[at:at + n]]).float().to(DEV).contiguous()
        o = run(step, state, i32(0, n, n + pad, 2 * n + pad), slots).cpu().double()
        outs[0].append(o[:n])
        outs[1].append(o[n + pad:])
        at += n
    assert float((state[[s for s in range(5) if s not in slot_of]] - 7.0).abs().max()) == 0.0, "another slot's state was touched"
    return [torch.cat(o) for o in outs], state


SIZES = [(3, 24, 40), (2, 80, 8), (4, 64, 64), (1, 5, 3), (2, 130, 16), (3, 256, 20), (1, 16, 128), (20, 64, 64), (2, 300, 7)]


@pytest.mark.parametrize("H,d,dv", SIZES)
def test_bonus_scan_reads_before_it_writes_and_carries_its_state(H, d, dv):
    """Some channels hardly decay, the bonus is far from 1: a read-out after the write, or a bonus that stays in
    the state, shows at once. Steps of 37, 1, 2, 17 and 6 tokens in slots out of order."""
    from llama_rs_metal_b200.kernels import ops
    gen = torch.Generator().manual_seed(H * 1000 + d)
    lengths = [37, 1, 2, 17, 6]
    n = sum(lengths)
    rand = lambda *s: torch.randn(*s, generator=gen, dtype=F64)  # noqa: E731
    bonus = rand(H, d) * 2.0
    seqs = [dict(r=rand(n, H, d), k=rand(n, H, d) * 0.5, v=rand(n, H, dv), w=torch.exp(-torch.exp(rand(n, H, d) - 1.0))) for _ in range(2)]
    for s in seqs:
        s["w"][:, :, 0] = 0.9999
    want = [P.bonus_scan(s["r"], s["k"], s["v"], s["w"], bonus) for s in seqs]

    def run(step, state, cu, slots):
        T, gap = step["r"].shape[0], 4
        proj = torch.zeros(T, gap + 2 * H * d + H * dv + 4, dtype=torch.float32, device=DEV)
        offs = dict(r=gap, v=gap + H * d, k=gap + H * d + H * dv)          # columns of a wider activation, in any order
        for name, o in offs.items():
            width = step[name].reshape(T, -1).shape[1]
            proj[:, o:o + width] = step[name].reshape(T, -1)
        return ops.bonus_state_scan(proj, offs["r"], offs["k"], offs["v"], step["w"].reshape(T, -1).contiguous(),
                                    bonus.float().to(DEV), state, cu, slots, dv)
    parts = {name: (seqs[0][name], seqs[1][name]) for name in "rkvw"}
    got, state = carried(parts, run, lengths, (H, d, dv), [3, 1])
    for b, s in enumerate(seqs):
        assert worst(got[b], want[b]) <= 3e-5, f"sequence {b}"
        S = torch.zeros(H, d, dv, dtype=F64)
        for t in range(n):
            S = s["w"][t][:, :, None] * S + s["k"][t][:, :, None] * s["v"][t][:, None, :]
        assert worst(state[[3, 1][b]], S) <= 3e-5


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 24, 40), (2, 2, 80, 8), (4, 1, 64, 64), (1, 1, 5, 3), (2, 1, 130, 16), (6, 3, 128, 20),
                                      (20, 20, 128, 128)])
def test_delta_scan_with_one_decay_per_head(H, G, d, dv):
    """A head that hardly decays and large step sizes: a decay after the removal, or a read-out ahead of the
    write, shows at once."""
    from llama_rs_metal_b200.kernels import ops
    gen = torch.Generator().manual_seed(H * 1000 + d + 7)
    lengths = [37, 1, 2, 17, 6]
    n = sum(lengths)
    rand = lambda *s: torch.randn(*s, generator=gen, dtype=F64)  # noqa: E731
    seqs = []
    for _ in range(2):
        g = torch.exp(-torch.exp(rand(n, H) - 1.0))
        g[:, 0] = 0.9999
        seqs.append(dict(q=P.unit_vector(rand(n, G, d)), k=P.unit_vector(rand(n, G, d)), v=rand(n, H, dv), g=g,
                         b=torch.sigmoid(rand(n, H) * 2.0)))
    wide = lambda x: x.repeat_interleave(H // G, dim=1)  # noqa: E731
    want = [P.delta_scan(wide(s["q"]), wide(s["k"]), s["v"], s["g"], s["b"]) for s in seqs]

    def run(step, state, cu, slots):
        return ops.head_decay_delta_scan(step["q"], step["k"], step["v"], step["g"], step["b"], state, cu, slots)
    got, _ = carried({name: (seqs[0][name], seqs[1][name]) for name in "qkvgb"}, run, lengths, (H, d, dv), [4, 0])
    for b in range(2):
        assert worst(got[b], want[b]) <= 3e-5, f"sequence {b}"


def portions(sequences, cuts, tail_shape, call):
    """Feed two sequences [n, W] in portions given as (tokens of the first, tokens of the second) with a sequence
    of padding between them; the tails of the slots used start at zero. -> results per sequence, tails."""
    tails = torch.full((4, *tail_shape), 3.0, dtype=torch.float32, device=DEV)
    tails[[2, 0]] = 0.0
    at, got, pad = [0, 0], [[], []], 3
    for n0, n1 in cuts:
        a, b = sequences[0][at[0]:at[0] + n0], sequences[1][at[1]:at[1] + n1]
        one_each = n0 == n1 == 1
        if one_each:
            x, cu, slots = torch.cat([a, b]), i32(0, 1, 2), i32(2, 0)
            seq_of = i32(0, 1)
        else:
            x = torch.cat([a, torch.ones(pad, a.shape[1], dtype=a.dtype), b])
            cu, slots = i32(0, n0, n0 + pad, n0 + pad + n1), i32(2, -1, 0)
            seq_of = i32(*([0] * n0 + [1] * pad + [2] * n1))
        out = call(x.to(DEV).contiguous(), tails, cu, seq_of, slots, one_each)
        skip = 0 if one_each else pad
        for i, t in enumerate(out if isinstance(out, tuple) else (out,)):
            got[0].append((i, t[..., :n0, :].cpu() if t.dim() == 3 and t.shape[1] == x.shape[0] and t.shape[0] != x.shape[0] else t[:n0].cpu()))
            got[1].append((i, t[..., n0 + skip:, :].cpu() if t.dim() == 3 and t.shape[1] == x.shape[0] and t.shape[0] != x.shape[0]
                           else t[n0 + skip:].cpu()))
        at = [at[0] + n0, at[1] + n1]
    assert float((tails[[1, 3]] - 3.0).abs().max()) == 0.0, "another slot's tail was touched"

    def joined(b, i, dim=0):
        return torch.cat([t for j, t in got[b] if j == i], dim=dim)
    return joined, tails


CUTS = [(1, 2), (5, 1), (1, 1), (1, 1), (17, 6), (1, 1), (2, 3)]     # 28 and 15 tokens


@pytest.mark.parametrize("n", [1, 2, 4, 7])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_delta_inputs_in_portions(n, dtype):
    from llama_rs_metal_b200.kernels import ops
    H, G, d, dv, gap = 4, 2, 20, 70, 3
    C = 2 * G * d + H * dv
    gen = torch.Generator().manual_seed(n)
    W = gap + C + 2 * H
    seqs = [(torch.randn(k, W, generator=gen) * 1.5).to(dtype) for k in (28, 15)]
    taps = torch.randn(n, C, generator=gen)
    rate, dt = torch.exp(torch.randn(H, generator=gen) - 1.0), torch.randn(H, generator=gen)

    def call(x, tails, cu, seq_of, slots, one_each):
        return ops.head_decay_delta_prepare(x, gap, gap + C, gap + C + H, dt.to(DEV), rate.to(DEV), taps.to(DEV),
                                            tails if n > 1 else None, cu, seq_of, slots, H, G, d, dv, 1e-6, d ** -0.5, one_each)
    joined, tails = portions(seqs, CUTS, (max(n - 1, 1), C), call)
    for b, s in enumerate(seqs):
        x = s.double()
        conv = P.silu(P.causal_conv(x[:, gap:gap + C], taps.double().t()))
        T = x.shape[0]
        want = [P.unit_vector(conv[:, :G * d].reshape(T, G, d)) * d ** -0.5, P.unit_vector(conv[:, G * d:2 * G * d].reshape(T, G, d)),
                conv[:, 2 * G * d:].reshape(T, H, dv),
                torch.exp(-rate.double() * P.softplus(x[:, gap + C + H:] + dt.double())), torch.sigmoid(x[:, gap + C:gap + C + H])]
        for i, w in enumerate(want):
            assert worst(joined(b, i), w) < 3e-6, (b, i)
        if n > 1:
            assert torch.equal(tails[[2, 0][b]].cpu(), s[-(n - 1):, gap:gap + C].float())


# --------------------------------------------------------------------------- convolution, norms, mixes
@pytest.mark.parametrize("n", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("dtype,W", [(torch.float32, 72), (torch.bfloat16, 72), (torch.bfloat16, 75), (torch.bfloat16, 1030)])
def test_input_convolution_alone_and_in_one_pass_with_the_norm(n, dtype, W):
    from llama_rs_metal_b200.kernels import ops
    gen = torch.Generator().manual_seed(n + W)
    taps = torch.randn(n, W, generator=gen)
    seqs = [torch.randn(k, W, generator=gen).to(dtype) for k in (28, 15)]
    tol = 1e-6 if dtype == torch.float32 else 6e-3

    def alone(x, tails, cu, seq_of, slots, one_each):
        return ops.input_conv(x, taps.to(DEV), tails if n > 1 else None, cu, seq_of, slots)
    joined, tails = portions(seqs, CUTS, (max(n - 1, 1), W), alone)
    for b, s in enumerate(seqs):
        assert worst(joined(b, 0), s.double() + P.causal_conv(s.double(), taps.double().t())) < tol
        if n > 1:
            assert torch.equal(tails[[2, 0][b]].cpu(), s[-(n - 1):].float())
    if n == 1:
        return
    # the stream's rows [float32] through the norm and the convolution, one pass where every sequence
    # brings one token, two where not, from the same tails; in the one-pass steps with slices to add
    g = 1.0 + 0.2 * torch.randn(W, generator=gen)
    streams = [torch.randn(k, W, generator=gen) * 3.0 + 1.0 for k in (28, 15)]
    written = []

    def both(x, tails, cu, seq_of, slots, one_each):
        if not one_each:
            return ops.input_conv(ops.layer_norm(x, g.to(DEV), None, 1e-5, dtype), taps.to(DEV), tails, cu, seq_of, slots)
        slices = torch.stack([0.25 * x, 0.5 * x, 0.125 * x])
        hidden = (0.125 * x).contiguous()
        out = ops.layer_norm_conv(hidden, g.to(DEV), None, 1e-5, dtype, taps.to(DEV), tails, slots, partials=slices)
        written.append(float((hidden - x).abs().max() / x.abs().max()))
        return out
    joined, tails = portions(streams, CUTS, (n - 1, W), both)
    assert len(written) == 3 and max(written) < 1e-6
    for b, s in enumerate(streams):
        h = P.layer_norm(s.double(), g.double(), 1e-5)
        assert worst(joined(b, 0), h + P.causal_conv(h, taps.double().t())) < (3e-6 if dtype == torch.float32 else 1.5e-2)


@pytest.mark.parametrize("W", [24, 75, 256, 1030, 4096, 8192, 9000])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_layer_norm_without_a_bias_adds_slices_first(W, dtype):
    from llama_rs_metal_b200.kernels import ops
    gen = torch.Generator().manual_seed(W)
    x = torch.randn(7, W, generator=gen) * 2.0 + 5.0          # a mean that a norm without centring would keep
    g, slices = 1.0 + 0.2 * torch.randn(W, generator=gen), torch.randn(3, 7, W, generator=gen)
    tol = 3e-6 if dtype == torch.float32 else 6e-3
    for planes in (None, slices):
        summed = x.double() + (planes.double().sum(0) if planes is not None else 0.0)
        hidden = x.clone().to(DEV)
        got = ops.layer_norm(hidden, g.to(DEV), None, 1e-5, dtype, partials=planes.to(DEV) if planes is not None else None)
        assert worst(got, P.layer_norm(summed, g.double(), 1e-5)) < tol
        assert worst(hidden, summed) < 1e-6
        rows = i32(5, 0)
        got = ops.layer_norm(x.clone().to(DEV), g.to(DEV), None, 1e-5, dtype, rows=rows, partials=planes.to(DEV) if planes is not None else None)
        assert worst(got, P.layer_norm(summed, g.double(), 1e-5)[[5, 0]]) < tol


@pytest.mark.parametrize("dtype,W", [(torch.float32, 72), (torch.bfloat16, 75), (torch.bfloat16, 1032)])
def test_token_mixes_read_the_row_before_and_keep_the_last(dtype, W):
    from llama_rs_metal_b200.kernels import ops
    gen = torch.Generator().manual_seed(W)
    mix = torch.rand(5, W, generator=gen)
    seqs = [torch.randn(k, W, generator=gen).to(dtype) for k in (28, 15)]

    def call(x, last, cu, seq_of, slots, one_each):
        return ops.token_mixes(x, mix.to(DEV), last, cu, seq_of, slots)
    joined, last = portions(seqs, CUTS, (1, W), call)
    for b, s in enumerate(seqs):
        h = s.double()
        before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
        want = torch.stack([h + (before - h) * m for m in mix.double()])
        assert worst(joined(b, 0, dim=1), want) < (1e-6 if dtype == torch.float32 else 6e-3)
        assert torch.equal(last[[2, 0][b], 0].cpu(), s[-1].float())


@pytest.mark.parametrize("T,N,K", [(1, 30, 5), (8, 128, 16), (70, 200, 64), (130, 96, 65), (3, 33, 130)])
def test_decay_product(T, N, K):
    from llama_rs_metal_b200.kernels import ops
    gen = torch.Generator().manual_seed(T + N)
    for gap in (0, 3, 8):
        proj = torch.randn(T, gap + K + gap, generator=gen) * 1.5
        w, bias = torch.randn(N, K, generator=gen) * K ** -0.5, torch.randn(N, generator=gen) - 2.0
        want = torch.exp(-torch.exp(torch.tanh(proj[:, gap:gap + K].double()) @ w.double().t() + bias.double()))
        assert worst(ops.decay_product(proj.to(DEV), gap, w.to(DEV), bias.to(DEV)), want) < 3e-6
        wb = w.bfloat16()
        want = torch.exp(-torch.exp(torch.tanh(proj[:, gap:gap + K].double()).bfloat16().double() @ wb.double().t() + bias.double()))
        assert worst(ops.decay_product(proj.to(DEV), gap, wb.to(DEV), bias.to(DEV)), want) < 2e-3   # a tanh may round the other way


# --------------------------------------------------------------------------- grouped products
@pytest.mark.parametrize("T", [1, 7, 8, 12, 40, 64, 65, 200, 700])
@pytest.mark.parametrize("K,group,last", [(64, 128, 16), (200, 256, 64), (72, 128, 5), (75, 128, 30), (512, 768, 16), (256, 512, 512)])
def test_grouped_products_multiply_each_input_with_its_own_rows(T, K, group, last):
    """Inputs of very different size, so that a row of a neighbouring input shows; every kernel that takes them."""
    from llama_rs_metal_b200.kernels import gemm_dispatch, ops
    gen = torch.Generator().manual_seed(T + K)
    G = 5
    x = torch.randn(G, T, K, generator=gen) * torch.tensor([1.0, 10.0, 0.1, 100.0, 3.0])[:, None, None]
    w = torch.randn(4 * group + last, K, generator=gen)
    xb, wb = x.bfloat16(), w.bfloat16()

    def reference(a, b):
        return [a[i].double() @ b[i * group:(i + 1) * group].double().t() for i in range(G)]

    def compare(got, want, tol, what):
        for i, r in enumerate(want):
            assert worst(got[:, i * group:i * group + r.shape[1]], r) < tol, f"{what}, input {i}"
    if T <= 200:
        compare(ops.linear_grouped(x.to(DEV), w.to(DEV), group), reference(x, w), 1e-5, "float32")
    want = reference(xb, wb)
    for pin in (None, 128, 256, 512, "pair"):
        gemm_dispatch.umma_width = pin
        try:
            compare(ops.linear_grouped(xb.to(DEV), wb.to(DEV), group), want, 1e-4, f"bfloat16, tile {pin}")
        finally:
            gemm_dispatch.umma_width = None
    gemm_dispatch.force_tiled = True
    try:
        compare(ops.linear_grouped(xb.to(DEV), wb.to(DEV), group), want, 1e-4, "bfloat16, warp-level")
    finally:
        gemm_dispatch.force_tiled = False
    gemm_dispatch.check_status()


# --------------------------------------------------------------------------- shaped heads, read-out, join, cap
@pytest.mark.parametrize("d,dv,rot,adjacent,bias,extra", [
    (12, 20, 6, False, False, 7), (64, 64, 64, False, False, 40), (96, 96, 32, False, True, 0), (128, 128, 128, True, False, 2),
    (10, 6, 2, True, True, 3), (15, 9, 4, False, False, 1), (200, 40, 0, False, False, 5), (300, 10, 20, False, True, 0)])
def test_head_norms_ahead_of_the_rotation(d, dv, rot, adjacent, bias, extra):
    """Weights per head dimension, rows longer than q | k | v, positions far from zero, with the angles from
    the step's table and made in the kernel; both kernels (heads of more than 256 take the general one)."""
    from llama_rs_metal_b200.kernels import ops
    Hq, Hk, T, base = 4, 2, 33, 50.0
    gen = torch.Generator().manual_seed(d)
    W = Hq * d + Hk * (d + dv)
    proj = torch.randn(T, W + extra, generator=gen)
    b = torch.randn(W, generator=gen) if bias else None
    qw, kw = 1.0 + 0.4 * torch.randn(d, generator=gen), 1.0 + 0.4 * torch.randn(d, generator=gen)
    positions = torch.arange(900, 900 + T)
    inv = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=F64) if rot else None
    x = proj[:, :W].double() + (b.double() if bias else 0.0)
    q = P.unit_rms(x[:, :Hq * d].reshape(T, Hq, d), 1e-5) * qw.double()
    k = P.unit_rms(x[:, Hq * d:(Hq + Hk) * d].reshape(T, Hk, d), 1e-5) * kw.double()
    v = x[:, (Hq + Hk) * d:].reshape(T, Hk, dv)
    if rot:
        if adjacent:      # neighbours: reorder to halves, turn, and back
            order = list(range(0, rot, 2)) + list(range(1, rot, 2)) + list(range(rot, d))
            back = torch.argsort(torch.tensor(order))
            q, k = (P.rotate_halves(t[..., order], positions, dict(dims=rot, base=base))[..., back] for t in (q, k))
        else:
            q, k = (P.rotate_halves(t, positions, dict(dims=rot, base=base)) for t in (q, k))
    pos = positions.to(torch.int32).to(DEV)
    for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 6e-3)):
        for table in (False, True):
            if table and not rot:
                continue
            args = dict(bias=b.to(DEV) if bias else None, head_weights=(qw.to(DEV), kw.to(DEV)), head_weight_eps=1e-5, rotary=rot,
                        adjacent_pairs=adjacent, inv_freq=inv.to(DEV) if rot else None)
            if table:
                args["table"] = ops.rope_table64(pos, inv.to(DEV))
            got = ops.shaped_qkv_store(proj.to(DEV), Hq, Hk, d, dv, pos, dtype, **args)
            for have, want in zip(got, (q, k, v)):
                assert worst(have, want) < tol


@pytest.mark.parametrize("H,dv", [(3, 20), (2, 64), (4, 100), (1, 256), (2, 300)])
def test_read_out_norm_into_columns(H, dv):
    from llama_rs_metal_b200.kernels import ops
    gen = torch.Generator().manual_seed(dv)
    T = 9
    o, gate, w = torch.randn(T, H, dv, generator=gen), torch.randn(T, 5 + H * dv, generator=gen), torch.randn(H * dv, generator=gen)
    want = P.unit_rms(o.double(), 1e-5).reshape(T, -1) * w.double() * P.silu(gate.double()[:, 5:]) * 0.6
    for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 6e-3)):
        wide = torch.full((T, 4 + H * dv + 3), 2.0, dtype=dtype, device=DEV)
        ops.head_norm_gate(o.to(DEV), 1e-5, dtype, weight=w.to(DEV), gate=gate.to(DEV), gate_column=5, gate_act=ops.GATE_SILU,
                           out_scale=0.6, out=wide, out_column=4)
        assert worst(wide[:, 4:-3], want) < tol
        assert float((wide[:, :4] - 2).abs().max()) == 0.0 and float((wide[:, -3:] - 2).abs().max()) == 0.0


def test_stream_swap_and_softcap():
    from llama_rs_metal_b200.kernels import ops
    gen = torch.Generator().manual_seed(1)
    x, base, planes = torch.randn(7, 40, generator=gen), torch.randn(7, 40, generator=gen), torch.randn(2, 7, 40, generator=gen)
    for dtype, tol in ((torch.float32, 1e-6), (torch.bfloat16, 5e-3)):
        for p in (None, planes):
            hidden = x.clone().to(DEV)
            out = ops.stream_swap_(hidden, base.to(DEV), dtype, p.to(DEV) if p is not None else None)
            assert torch.equal(hidden.cpu(), base)
            assert worst(out, x.double() + (p.double().sum(0) if p is not None else 0.0)) < tol
    z = torch.randn(5, 33, generator=gen) * 30.0
    assert worst(ops.softcap_(z.clone().to(DEV), 7.0), P.softcap(z.double(), 7.0)) < 1e-6
