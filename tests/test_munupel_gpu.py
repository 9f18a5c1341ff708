"""The Munupel decoder on the GPU against the plain float64 implementation (tests/plain_munupel.py): whole
models through the step function, the cache and the generation loop. Its mechanisms alone are in
test_munupel_mechanisms_gpu.py."""
import numpy as np
import pytest
import torch

import helpers
import plain_munupel as P

pytestmark = pytest.mark.gpu
F64 = torch.float64
NAMES = ["M1", "M2", "M3"]


@pytest.fixture(scope="module")
def engine():
    from llama_rs_metal_b200 import Engine
    return Engine()


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("munupel")
    return {name: helpers.make_munupel_dir(str(root / name), name) for name in NAMES}


@pytest.fixture(scope="module")
def plain(folders):
    return {name: P.read_model(path) for name, path in folders.items()}


_REFS = {}


def reference(plain, name, tokens):
    key = (name, tuple(tokens))
    if key not in _REFS:
        config, tensors = plain[name]
        _REFS[key] = P.forward(config, tensors, tokens).numpy()
    return _REFS[key]


# Allowed error of a row of logits as a fraction of the largest reference logit. float32: sums in
# another order than the plain implementation's float64.
# bfloat16: activations are rounded between kernels; a fault of any mechanism is far above. In bfloat16
# one row in twenty may be up to four times over while the median stays below a third.
TOLERANCE = {"float32": 2e-5, "bfloat16": 5e-2}


def close(got, ref, dtype, what, factor=1.0):
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    if ref.ndim == 1:
        got, ref = got.reshape(1, -1), ref.reshape(1, -1)
    assert got.shape == ref.shape and np.all(np.isfinite(got)), what
    err = np.abs(got - ref).max(axis=-1) / max(float(np.abs(ref).max()), 1e-30)
    allowed = factor * TOLERANCE[dtype]
    worst = int(err.argmax())
    report = (f"{what}: row {worst} off by {err[worst]:.3e} of the largest logit (allowed {allowed:.0e}); first such row "
              f"{int(np.argmax(err > allowed))}; {int((err > allowed).sum())} of {len(err)} rows over; median {np.median(err):.3e}")
    if dtype == "bfloat16" and len(err) >= 8:
        assert (err > allowed).sum() <= max(1, len(err) // 20) and err[worst] <= 4 * allowed \
            and np.median(err) <= allowed / 3, report
    else:
        assert err[worst] <= allowed, report


def vocab_of(name):
    return helpers.MUNUPEL[name]["config"]["vocab"]


def open_runner(engine, folder, dtype, max_tokens=2048, max_slots=8, use_graphs=True):
    from llama_rs_metal_b200.cache import Cache
    from llama_rs_metal_b200.engine.session import build_model
    from llama_rs_metal_b200.engine.step import StepRunner
    from llama_rs_metal_b200.runtime import Runtime, parse_dtype
    rt = Runtime(engine.device, parse_dtype(dtype))
    _, _, model, _ = build_model(folder, rt)
    cache = Cache(model.cache_requests(), rt.dtype, rt.device, max_tokens, max_slots, max_tokens)
    return StepRunner(model, cache, rt, use_graphs=use_graphs), cache, model


def entry(slot, tokens, want=None):
    from llama_rs_metal_b200.engine.batch import StepEntry
    return StepEntry(slot, tokens, range(len(tokens)) if want is None else want)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_match_the_plain_implementation(engine, folders, plain, name, dtype):
    runner, cache, _ = open_runner(engine, folders[name], dtype)
    for i, n in enumerate([150, 37, 1, 2, 3]):    # the first tokens of a sequence are rows 0, 1, ...
        tokens = helpers.random_tokens(300 + i, n, vocab_of(name))
        slot = cache.open_slot()
        got = runner.step([entry(slot, tokens)]).cpu().numpy()
        cache.close_slot(slot)                     # the next prompt takes the same slot and state
        close(got, reference(plain, name, tokens), dtype, f"{name} prompt of {n}")
    runner.check_device_status()


@pytest.mark.parametrize("name", NAMES)
def test_every_layer_matches_the_plain_residual_stream(engine, folders, plain, name):
    runner, cache, model = open_runner(engine, folders[name], "float32", use_graphs=False)
    seen = []
    for block in model.blocks:
        def wrapped(hidden, ctx, view, inner=block.forward):
            out = inner(hidden, ctx, view)
            seen.append(out.detach().clone().cpu().to(F64))
            return out
        block.forward = wrapped
    tokens = helpers.random_tokens(8, 90, vocab_of(name))
    runner.step([entry(cache.open_slot(), tokens, [])])
    config, tensors = plain[name]
    streams = []
    P.forward(config, tensors, tokens, streams)
    assert len(seen) == len(streams) == len(config["layers"])
    for i, (got, want) in enumerate(zip(seen, streams)):
        err = float((got[:len(tokens)] - want).abs().max() / want.abs().max())
        assert err < 2e-5, f"{name}: the stream after layer {i} is off by {err:.2e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_prefill_then_decoding_in_an_unequal_batch(engine, folders, plain, name, dtype):
    """Prompts of unequal lengths in one step, then one token each per step, past a page's border and past
    every window; the shorter requests end earlier and the batch shrinks."""
    runner, cache, _ = open_runner(engine, folders[name], dtype)
    V = vocab_of(name)
    totals, prompts = [140, 75, 9, 58], [100, 60, 1, 2]
    seqs = [helpers.random_tokens(40 + i, n, V) for i, n in enumerate(totals)]
    refs = [reference(plain, name, s) for s in seqs]
    slots = [cache.open_slot() for _ in seqs]
    out = runner.step([entry(sl, s[:n]) for sl, s, n in zip(slots, seqs, prompts)]).cpu().numpy()
    row = 0
    for b, n in enumerate(prompts):
        close(out[row:row + n], refs[b][:n], dtype, f"{name} prompt {b} in the batch")
        row += n
    at, decoded = list(prompts), [[] for _ in seqs]
    while any(a < t for a, t in zip(at, totals)):
        live = [b for b in range(len(seqs)) if at[b] < totals[b]]
        out = runner.step([entry(slots[b], [seqs[b][at[b]]]) for b in live]).cpu().numpy()
        for i, b in enumerate(live):
            decoded[b].append(out[i])
            at[b] += 1
            if at[b] == totals[b]:
                cache.close_slot(slots[b])
    for b, n in enumerate(prompts):
        close(np.stack(decoded[b]), refs[b][n:], dtype, f"{name} sequence {b}, decoded from position {n}")
    runner.check_device_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["M1", "M2"])
def test_a_prompt_geometry_that_comes_again_is_captured_and_replayed(engine, folders, plain, name, dtype):
    """The same shape of batch four times with other tokens, in slots and pages that were used before, also under
    a captured graph's replay."""
    runner, cache, _ = open_runner(engine, folders[name], dtype)
    V = vocab_of(name)
    following, expected = [], []
    for turn in range(4):
        seqs = [helpers.random_tokens(500 + 10 * turn + i, n, V) for i, n in enumerate([70, 3, 41])]
        slots = [cache.open_slot() for _ in seqs]
        out = runner.step([entry(sl, s) for sl, s in zip(slots, seqs)]).cpu().numpy()
        row = 0
        for s in seqs:
            close(out[row:row + len(s)], reference(plain, name, s), dtype, f"{name} turn {turn}")
            row += len(s)
        nxt = [int(t) for t in helpers.random_tokens(900 + turn, len(seqs), V)]
        out = runner.step([entry(sl, [t]) for sl, t in zip(slots, nxt)]).cpu().numpy()
        for i, (s, t) in enumerate(zip(seqs, nxt)):
            following.append(out[i])
            expected.append(reference(plain, name, s + [t])[-1])
        for sl in slots:
            cache.close_slot(sl)
    close(np.stack(following), np.stack(expected), dtype, f"{name}: the token after each prompt")
    runner.check_device_status()


@pytest.mark.parametrize("sizes", [[2], [3, 64, 5], [1, 70, 2], [64], [17]])
@pytest.mark.parametrize("name", ["M1", "M2"])
def test_portions_of_any_size_give_the_whole_prompt(engine, folders, plain, name, sizes):
    for dtype in ("float32", "bfloat16"):
        runner, cache, _ = open_runner(engine, folders[name], dtype)
        tokens = helpers.random_tokens(77, 150 if sizes != [2] else 40, vocab_of(name))
        ref = reference(plain, name, tokens)
        slot, at, i, rows = cache.open_slot(), 0, 0, []
        while at < len(tokens):
            n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
            rows.append(runner.step([entry(slot, tokens[at:at + n])]).cpu().numpy())
            at, i = at + n, i + 1
        close(np.concatenate(rows), ref, dtype, f"{name} in portions of {sizes}")
        cache.close_slot(slot)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_company_in_the_batch_changes_nothing_beyond_rounding(engine, folders, plain, dtype):
    name = "M2"
    runner, cache, _ = open_runner(engine, folders[name], dtype)
    V = vocab_of(name)
    mine = helpers.random_tokens(5, 130, V)
    others = [helpers.random_tokens(6 + i, n, V) for i, n in enumerate([200, 3, 64])]
    slot = cache.open_slot()
    alone = runner.step([entry(slot, mine)]).cpu().numpy()
    cache.close_slot(slot)
    slots = [cache.open_slot() for _ in range(4)]
    together = runner.step([entry(slots[0], others[0], []), entry(slots[1], mine), entry(slots[2], others[1], []),
                            entry(slots[3], others[2], [])]).cpu().numpy()
    limit = 1e-5 if dtype == "float32" else 3e-2
    assert np.abs(alone - together).max() <= limit * np.abs(alone).max()
    close(together, reference(plain, name, mine), dtype, "in company")


def test_a_freed_slot_and_its_pages_start_from_nothing(engine, folders, plain):
    """The pages a sequence gave back, those of its first tokens among them, hold another sequence's keys when
    they are used again."""
    name = "M1"
    for dtype in ("float32", "bfloat16"):
        runner, cache, _ = open_runner(engine, folders[name], dtype, max_tokens=512, max_slots=2)
        V = vocab_of(name)
        slot = cache.open_slot()
        runner.step([entry(slot, helpers.random_tokens(1, 200, V), [])])
        for t in helpers.random_tokens(2, 5, V):
            runner.step([entry(slot, [t], [])])
        cache.close_slot(slot)
        second = helpers.random_tokens(3, 90, V)
        again = cache.open_slot()
        assert again == slot
        got = [runner.step([entry(again, second[:50])]).cpu().numpy()]
        for t in second[50:]:
            got.append(runner.step([entry(again, [t])]).cpu().numpy())
        close(np.concatenate(got), reference(plain, name, second), dtype, "the slot's second sequence")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["M1", "M2"])
def test_long_decoding_through_captured_steps(engine, folders, plain, name, dtype):
    """300 tokens one by one from the very first through captured steps: pages, windows and chunks pass by, the
    first tokens stay."""
    runner, cache, _ = open_runner(engine, folders[name], dtype)
    tokens = helpers.random_tokens(9, 300, vocab_of(name))
    slot = cache.open_slot()
    rows = [runner.step([entry(slot, [t])]).cpu().numpy() for t in tokens]
    close(np.concatenate(rows), reference(plain, name, tokens), dtype, "token by token from the start", factor=2.0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_session(engine, folders, plain, dtype):
    from llama_rs_metal_b200 import GenerationOptions, Sampling
    name = "M2"
    model = engine.load(folders[name], dtype=dtype)
    session = model.session(context=256, max_batch=4)
    V = vocab_of(name)
    prompts = [helpers.random_tokens(60 + i, n, V) for i, n in enumerate([70, 5, 33])]
    results = session.generate(prompts, GenerationOptions(max_tokens=12, sampling=Sampling(temperature=0.0)))
    config, tensors = plain[name]
    for prompt, result in zip(prompts, results):
        tokens = list(prompt)
        assert len(result.tokens) == 12
        for chosen in result.tokens:
            logits = P.forward(config, tensors, tokens)[-1].numpy()
            best = int(logits.argmax())
            if chosen != best:   # a near tie may fall the other way under rounding
                gap = (logits[best] - logits[chosen]) / np.abs(logits).max()
                assert gap < (1e-4 if dtype == "float32" else 5e-2), f"chose {chosen}, the plain model {best} by {gap:.2e}"
            tokens.append(chosen)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_through_the_trace_runner(folders, plain, dtype, tmp_path):
    name = "M1"
    V = vocab_of(name)
    requests = {f"r{i}": helpers.random_tokens(90 + i, n, V) for i, n in enumerate([120, 40, 77])}
    trace = helpers.Trace()
    trace.whole("whole:r0", requests["r0"])
    trace.tail_one_by_one("tail:r1", requests["r1"], tail=20)
    trace.batch({f"batch:{n}": t for n, t in requests.items()}, {"batch:r0": 90, "batch:r1": 10, "batch:r2": 70})
    outputs = helpers.run_trace(folders[name], dtype, trace, 1024, str(tmp_path / "out"))
    refs = {n: reference(plain, name, t) for n, t in requests.items()}
    for step in sorted(trace.rows):
        rows = trace.rows[step]
        close(outputs[step], np.stack([refs[rid.split(":")[-1]][pos] for rid, pos in rows]), dtype, f"step {step}")


def test_sublayers_are_joined_under_bfloat16_only(engine, folders, tmp_path):
    """Layers with a feed-forward run as two products; in float32, and where rows are no whole 16-byte pieces, as
    they are."""
    odd = dict(config=dict(architecture="Munupel", vocab=50, width=60, norm=dict(eps=1e-5), layers=[
        helpers._window_layer(helpers._gated(2, 1, 8, 12, 0.3, 5, keep_first=1), 32)]), seed=1, std=0.1)
    folder = helpers.make_munupel_dir(str(tmp_path), odd)
    for path, dtype, joined in ((folders["M2"], "bfloat16", [True] * 3), (folders["M1"], "bfloat16", [True, False]),
                                (folders["M2"], "float32", [False] * 3), (folder, "bfloat16", [False])):
        _, _, model = open_runner(engine, path, dtype)
        assert [b.into is not None for b in model.blocks if b.kind == "parallel"] == joined, (path, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_first_token_is_seen_by_layers_that_keep_it_and_by_no_others(engine, folders, dtype, tmp_path):
    """One windowed layer on its own, with a sequence's third token replaced far away: the logits move where the
    layer keeps three first keys, and do not move at all where it keeps two, in prompts and in decoding."""
    moved = {}
    for keep in (2, 3):
        spec = dict(config=dict(architecture="Munupel", vocab=128, width=64, norm=dict(eps=1e-5), layers=[
            helpers._window_layer(helpers._gated(4, 2, 32, 32, 0.3, 20, keep_first=keep), 64)]), seed=5, std=0.1)
        folder = helpers.make_munupel_dir(str(tmp_path / f"{keep}{dtype}"), spec)
        runner, cache, _ = open_runner(engine, folder, dtype)
        rows = []
        for third in (7, 90):
            tokens = helpers.random_tokens(3, 200, 128)
            tokens[2] = third
            slot = cache.open_slot()
            out = [runner.step([entry(slot, tokens[:180])])[150:]]
            out += [runner.step([entry(slot, [t])]) for t in tokens[180:]]
            cache.close_slot(slot)
            rows.append(torch.cat(out).cpu())
        moved[keep] = (rows[0] - rows[1]).abs().amax(dim=1)
    assert float(moved[2].max()) == 0.0 and float(moved[3].min()) > 1e-4


# --------------------------------------------------------------------------- configurations drawn at random
def drawn_configuration(seed):
    rng = np.random.default_rng(seed)

    def pick(*values):
        return values[int(rng.integers(len(values)))]
    width = int(pick(40, 64, 88, 136, 232))
    layers = []
    for _ in range(int(rng.integers(2, 6))):
        kv = int(pick(1, 2, 3))
        dim, heads = int(pick(4, 16, 24, 64, 96, 128)), kv * int(pick(1, 2, 3))
        rot = None
        if pick(True, True, True, False):
            scaling = pick(None, (8.0, 128, 32.0, 1.0), (2.0, 40, 3.0, 0.5), (4.0, 1000, 16.0, 2.0))
            rot = helpers._scaled_rotation(int(pick(*[r for r in (2, 4, 16, 24, 64, 96) if r <= dim])), float(pick(30.0, 10000.0, 200000.0)), scaling)
        sizes = (heads, kv, dim, int(pick(dim, 8, 12, 32, 96)), float(pick(0.1, 0.3)))
        ff = int(pick(24, 64, 100)) if rng.integers(3) else None
        if pick(True, False):
            layers.append(helpers._chunk_layer(helpers._gated(*sizes, pick(None, 1, 2, 33, 64, 90, 200), rot, pick(None, 2.0, 5.0)), ff))
        else:
            size = pick(None, 1, 2, 40, 64, 65, 130)
            layers.append(helpers._window_layer(helpers._gated(*sizes, size, rot, keep_first=pick(None, 1, 17, 64, 70) if size else None), ff))
    if rng.integers(3):
        of = int(rng.integers(len(layers)))
        layers.insert(int(rng.integers(of + 1, len(layers) + 1)), dict(layers[of], weights_of=of))
    return dict(config=dict(architecture="Munupel", vocab=int(pick(97, 256, 333)), width=width, norm=dict(eps=float(pick(1e-6, 1e-4))),
                            layers=layers), seed=5000 + seed, std=float(pick(0.08, 0.15)))


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(engine, tmp_path, seed):
    """Other sizes, orders of layers, owners of tensors and constants than the fixed configurations: a prompt whole,
    then tokens one by one, a second sequence beside it in portions."""
    spec = drawn_configuration(seed)
    folder = helpers.make_munupel_dir(str(tmp_path / "m"), spec)
    config, tensors = P.read_model(folder)
    V = spec["config"]["vocab"]
    a, b = helpers.random_tokens(seed, 150, V), helpers.random_tokens(seed + 50, 100, V)
    ref_a, ref_b = P.forward(config, tensors, a).numpy(), P.forward(config, tensors, b).numpy()
    for dtype in ("float32", "bfloat16"):
        runner, cache, _ = open_runner(engine, folder, dtype)
        sa, sb = cache.open_slot(), cache.open_slot()
        out = runner.step([entry(sa, a[:120]), entry(sb, b[:3])]).cpu().numpy()
        close(out[:120], ref_a[:120], dtype, f"seed {seed}: prompt a", factor=2.0)
        close(out[120:], ref_b[:3], dtype, f"seed {seed}: prompt b", factor=2.0)
        out = runner.step([entry(sa, a[120:121]), entry(sb, b[3:70])]).cpu().numpy()     # one token and a portion
        close(out[:1], ref_a[120:121], dtype, f"seed {seed}: a's next token", factor=2.0)
        close(out[1:], ref_b[3:70], dtype, f"seed {seed}: b's portion", factor=2.0)
        rows_a, rows_b = [], []
        for t in range(121, 150):
            entries = [entry(sa, [a[t]])] + ([entry(sb, [b[t - 51]])] if t - 51 < 100 else [])
            out = runner.step(entries).cpu().numpy()
            rows_a.append(out[0])
            if len(entries) > 1:
                rows_b.append(out[1])
        close(np.stack(rows_a), ref_a[121:], dtype, f"seed {seed}: a decoded", factor=2.0)
        close(np.stack(rows_b), ref_b[70:70 + len(rows_b)], dtype, f"seed {seed}: b decoded", factor=2.0)
        runner.check_device_status()
