"""The Munupel decoder without a GPU: configuration, plan, tensor names, cache requests, kept pages, and the plain
implementation's mechanisms against values worked out by hand."""
import json
import math

import numpy as np
import pytest
import torch

import helpers
import plain_munupel as P
from llama_rs_metal_b200.cache import Cache
from llama_rs_metal_b200.config.munupel import MunupelConfig
from llama_rs_metal_b200.engine.model import DecoderModel
from llama_rs_metal_b200.errors import CacheMemoryError, InvalidError, UnsupportedError
from llama_rs_metal_b200.parts.attention import Attention
from llama_rs_metal_b200.parts.base import KeyValueRequest, PartSpec
from llama_rs_metal_b200.parts.linear import SplitLinear
from llama_rs_metal_b200.parts.rope import RotaryEmbedding
from llama_rs_metal_b200.registry import find_architecture
from llama_rs_metal_b200.runtime import Runtime

F64 = torch.float64


def build(root):
    root = helpers.MUNUPEL[root]["config"] if isinstance(root, str) else root
    arch = find_architecture(root)
    config = arch.config_class.from_dict(root)
    return config, arch.plan(config)


def cpu_model(plan):
    return DecoderModel(plan, Runtime(torch.device("cpu"), torch.float32))


# --------------------------------------------------------------------------- configuration and plan
@pytest.mark.parametrize("name", sorted(helpers.MUNUPEL))
def test_configuration_reads_every_size_and_writes_it_back(name):
    config, _ = build(name)
    assert MunupelConfig.from_dict(config.to_dict()) == config
    assert len(config.layers) == len(helpers.MUNUPEL[name]["config"]["layers"])


def test_absent_options_are_off():
    _, plan = build("M3")
    full, last = plan.layers[0].parts["mixer"].params, plan.layers[-1].parts["mixer"].params
    assert full["position"] is None and full["chunk"] is None and full["score_cap"] is None
    assert last["chunk"] == 1 and last["score_cap"] == 2.0 and last["position"].params.get("scaling", "default") == "default"
    assert plan.layers[0].block == "parallel_mixer" and plan.layers[-1].block == "parallel"
    one = plan.layers[1].parts["mixer"].params
    assert one["window"] == 1 and one["keep_first"] == 0 and "score_cap" not in one


def test_configuration_names_what_is_missing_or_not_built():
    root = helpers.MUNUPEL["M2"]["config"]

    def changed(path, value):
        out = json.loads(json.dumps(root))               # (nothing shared between layers)
        at = out
        for key in path[:-1]:
            at = at[key]
        if value is None:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        return out
    mixer = ("layers", 1, "mixer")
    for path, value, word in [(("width",), None, "width"), (mixer + ("kv_heads",), 3, "multiple"), (mixer + ("scale",), None, "scale"),
                              (mixer + ("rot", "dims"), 42, "rot"), (mixer + ("rot", "dims"), 7, "rot"), (mixer + ("rot", "base"), None, "base"),
                              (mixer + ("rot", "scaling", "slow"), None, "slow"), (mixer + ("rot", "scaling", "factor"), 0.0, "positive"),
                              (mixer + ("softcap",), -1.0, "softcap"), (mixer + ("mask", "size"), 0, "size"), (mixer + ("vdim",), None, "vdim"),
                              (("norm", "eps"), None, "eps"), (("layers", 0, "mlp", "ff"), None, "ff"), (("layers",), [], "layers"),
                              (("layers", 2, "weights_of"), 9, "weights_of"), (("layers", 2, "weights_of"), 2, "weights_of"),
                              (("layers", 2, "weights_of"), 1, "differ"), (("layers", 2, "mixer", "scale"), 0.5, "differ")]:
        with pytest.raises(InvalidError, match=word):
            MunupelConfig.from_dict(changed(path, value))
    with pytest.raises(UnsupportedError, match="type"):
        MunupelConfig.from_dict(changed(("layers", 0, "type"), "attention_3"))
    with pytest.raises(UnsupportedError, match="kind"):
        MunupelConfig.from_dict(changed(("layers", 0, "mlp", "kind"), "moe"))


def test_a_layer_may_run_another_layers_tensors_on_a_cache_of_its_own():
    _, plan = build("M1")
    assert [(e.layer, e.cache) for e in plan.schedule] == [(0, 0), (1, 1), (2, 2), (0, 3), (3, 4)]
    _, plan = build("M3")            # layer 1 runs layer 3's, layer 4 what layer 1 runs
    assert [(e.layer, e.cache) for e in plan.schedule] == [(0, 0), (2, 1), (1, 2), (2, 3), (2, 4), (3, 5)]
    specs = cpu_model(plan).tensor_specs()
    assert "l3.mix.q" in specs and not any(n.startswith(("l1.", "l4.")) for n in specs)
    assert [P.tensors_of(helpers.MUNUPEL["M3"]["config"], i) for i in range(6)] == [0, 3, 2, 3, 3, 5]


def test_tensor_names_and_shapes():
    _, plan = build("M1")
    shapes = {name: spec.shape for name, spec in cpu_model(plan).tensor_specs().items()}
    assert shapes["embed"] == shapes["head"] == (211, 72)
    assert shapes["final.norm"] == shapes["final.norm.b"] == shapes["l0.norm1"] == shapes["l2.norm1.b"] == (72,)
    chunked = dict(q=(48, 72), k=(24, 72), v=(40, 72), g=(80, 72), o=(72, 80))
    chunked.update({"q.b": (48,), "k.b": (24,), "v.b": (40,), "o.b": (72,)})
    windowed = dict(q=(30, 72), k=(30, 72), v=(18, 72), g=(3, 72), o=(72, 18), sink=(3,))
    for prefix, own in (("l0.mix.", chunked), ("l1.mix.", windowed)):
        assert {n: s for n, s in shapes.items() if n.startswith(prefix)} == {prefix + n: s for n, s in own.items()}
    assert shapes["l0.mlp.gate"] == (56, 72) and "l1.mlp.gate" not in shapes and "l1.norm2" not in shapes


def test_cache_requests_keep_what_each_layer_needs():
    _, plan = build("M1")
    assert cpu_model(plan).cache_requests() == [
        KeyValueRequest(2, 12, 7, 20), KeyValueRequest(3, 10, 9, 6, keep_first=3), KeyValueRequest(2, 16, 40, 10, keep_first=1),
        KeyValueRequest(2, 12, 7, 20), KeyValueRequest(1, 18, 70)]
    _, plan = build("M3")            # without a mask everything is kept, and kept keys say nothing
    assert cpu_model(plan).cache_requests()[0] == KeyValueRequest(2, 16, None, 24)
    assert Attention(64, 2, 1, 16, gate="head", keep_first=9).cache_request() == KeyValueRequest(1, 16)


def test_stretched_frequencies_agree_with_the_position_encoding():
    for dims, base, scaling in ((32, 10000.0, (4.0, 256, 32.0, 1.0)), (24, 1e6, (8.0, 4096, 16.0, 2.0)), (6, 50.0, (8.0, 64, 4.0, 0.5)),
                                (64, 500.0, (3.0, 100000, 64.0, 8.0)), (10, 100.0, (2.0, 3, 500.0, 400.0)), (8, 30.0, None)):
        rot = helpers._scaled_rotation(dims, base, scaling)
        params = dict(scaling="yarn", factor=scaling[0], original_max_position_embeddings=scaling[1], fast_turns=scaling[2],
                      slow_turns=scaling[3]) if scaling else {}
        encoding = RotaryEmbedding(128, dims, base, **params)
        freqs, stretch = P.rotation(rot)
        assert np.allclose(encoding.inverse_frequencies(), freqs, rtol=1e-13) and abs(encoding.magnitude - stretch) < 1e-15
        if scaling:
            with pytest.raises(UnsupportedError, match="magnitude"):
                encoding.rotary_table()
    freqs, stretch = P.rotation(helpers._scaled_rotation(32, 10000.0, (4.0, 256, 32.0, 1.0)))
    ratio = np.array(freqs) / np.array(P.rotation(dict(dims=32, base=10000.0))[0])
    assert (ratio == 1).any() and np.isclose(ratio, 0.25).any() and ((ratio > 0.26) & (ratio < 0.99)).any()
    assert abs(stretch - (0.1 * math.log(4.0) + 1.0)) < 1e-15


def test_attention_options_that_exclude_each_other():
    with pytest.raises(InvalidError, match="gate"):
        Attention(64, 2, 1, 16, gate="row")
    with pytest.raises(InvalidError, match="cap"):
        Attention(64, 2, 1, 16, score_cap=0.0)
    with pytest.raises(InvalidError, match="softmax"):
        Attention(64, 2, 1, 16, weights="sigmoid", keep_first=4)
    with pytest.raises(InvalidError, match="shaped"):
        Attention(64, 2, 1, 16, score_cap=5.0, query_temperature=(0.1, 4))
    with pytest.raises(InvalidError, match="shaped"):
        Attention(64, 2, 1, 16, sinks=True, head_norm_eps=1e-5)
    assert Attention(64, 2, 1, 16, sinks=True, score_cap=5.0, value_dim=24).mixed_width == 48
    stretched = PartSpec("rope", dict(head_dim=16, rotary_dim=8, theta=100.0, scaling="yarn", factor=4.0, original_max_position_embeddings=64))
    assert Attention(64, 2, 1, 16, position=stretched).shaped and not Attention(64, 2, 1, 16).shaped


def test_two_products_with_one_input_divide_at_whole_pieces():
    plain, gate_up = torch.ones(70, 8), torch.full((32, 8), 2.0)
    both = SplitLinear(plain, gate_up)
    assert both.columns == 96 and tuple(both.weight.shape) == (128, 8)
    assert torch.equal(both.weight[:70], plain) and not both.weight[70:96].any() and torch.equal(both.weight[96:], gate_up)


# --------------------------------------------------------------------------- pages of kept first tokens
def kept_cache(window, keep, pages=6, slots=2, page_size=4):
    request = KeyValueRequest(1, 2, window, keep_first=keep)
    return Cache([request], torch.float32, torch.device("cpu"), pages * page_size, slots, 100, page_size=page_size)


def held(cache, slot):
    return [i for i, p in enumerate(cache.kv_groups[0].table_host[slot]) if p >= 0]


@pytest.mark.parametrize("keep,head", [(1, [0]), (4, [0]), (5, [0, 1]), (0, [])])
def test_pages_of_first_tokens_stay_while_the_window_moves_on(keep, head):
    cache = kept_cache(window=6, keep=keep, pages=12)
    slot = cache.open_slot()
    cache.grow([(slot, 5)])
    cache.commit([(slot, 5)])
    for n in range(5, 40):                                    # one token at a time
        before, rows = cache.grow_by_one(np.array([slot]))
        cache.commit_lengths(np.array([slot]), before + 1)
        seen = list(range(max(0, n + 1 - 6) // 4, n // 4 + 1))
        assert held(cache, slot) == sorted(set(head) & set(range(n // 4 + 1)) | set(seen)), n
        assert rows[0][0] == cache.kv_groups[0].table_host[slot, n // 4] * 4 + n % 4
    first = [int(p) for p in cache.kv_groups[0].table_host[slot, :len(head)]]
    cache.grow([(slot, 60, 40)])                               # a portion: what its first query sees stays
    cache.commit([(slot, 60)])
    assert held(cache, slot) == head + list(range((41 - 6) // 4, 15))
    assert [int(p) for p in cache.kv_groups[0].table_host[slot, :len(head)]] == first
    cache.close_slot(slot)
    assert cache.kv_groups[0].pool.held == 0


def test_a_long_prompt_keeps_its_first_pages_and_its_window_only():
    cache = kept_cache(window=6, keep=5, pages=5)
    slot = cache.open_slot()
    cache.grow([(slot, 50)])
    rows = cache.destination_rows([slot], [0], [50])[0]
    stored = [i for i, r in enumerate(rows) if r >= 0]
    assert stored == list(range(8)) + list(range(44, 50)) and len(set(rows[stored])) == len(stored)
    cache.commit([(slot, 50)])
    other = cache.open_slot()
    with pytest.raises(CacheMemoryError):                      # first pages count: two of its own and a window of two
        cache.grow([(other, 50)])
    assert held(cache, other) == []
    cache.grow([(other, 4)])


def test_sequences_share_nothing_of_their_first_pages():
    cache = kept_cache(window=6, keep=5, pages=9)
    a, b = cache.open_slot(), cache.open_slot()
    cache.grow([(a, 30), (b, 22)])
    cache.commit([(a, 30), (b, 22)])
    pages = [int(p) for s in (a, b) for p in cache.kv_groups[0].table_host[s] if p >= 0]
    assert len(pages) == len(set(pages)) == 8
    cache.close_slot(a)
    again = cache.open_slot()
    cache.grow([(again, 3)])
    assert held(cache, again) == [0] and held(cache, b)[:2] == [0, 1]


# --------------------------------------------------------------------------- the plain mechanisms by hand
def test_norm_and_cap_by_hand():
    x = torch.tensor([[1.0, 3.0]], dtype=F64)
    w, b = torch.tensor([2.0, 5.0], dtype=F64), torch.tensor([10.0, -1.0], dtype=F64)
    assert torch.allclose(P.layer_norm(x, w, b, 0.0), torch.tensor([[8.0, 4.0]], dtype=F64))
    assert torch.allclose(P.layer_norm(x, w, b, 3.0), torch.tensor([[9.0, 1.5]], dtype=F64))   # eps inside the root
    z = torch.tensor([1.0, 100.0], dtype=F64)
    assert torch.allclose(P.softcap(z, 2.0), torch.tensor([2.0 * math.tanh(0.5), 2.0], dtype=F64)) and torch.equal(P.softcap(z, None), z)


def test_which_keys_a_query_sees():
    assert P.chunk_sees(7, 4) == [4, 5, 6, 7] and P.chunk_sees(8, 4) == [8] and P.chunk_sees(2, 4) == [0, 1, 2]
    assert P.chunk_sees(3, None) == [0, 1, 2, 3] and P.chunk_sees(5, 1) == [5]
    assert P.window_sees(9, 3, 2) == [0, 1, 7, 8, 9] and P.window_sees(3, 3, 2) == [0, 1, 2, 3]
    assert P.window_sees(1, 1, 5) == [0, 1] and P.window_sees(9, 1, 0) == [9] and P.window_sees(2, None, 0) == [0, 1, 2]


def test_a_sink_takes_its_share_once_and_a_cap_bounds_a_score():
    T = 4
    q, k = torch.ones(T, 2, 1, dtype=F64), torch.zeros(T, 1, 1, dtype=F64)
    k[1] = 50.0
    v = torch.eye(T, dtype=F64).reshape(T, 1, T)
    sinks = torch.tensor([0.0, math.log(5.0)], dtype=F64)
    out = P.attention(q, k, v, 1.0, lambda i: list(range(i + 1)), cap=2.0, sinks=sinks)
    e = math.exp(2.0)
    assert torch.allclose(out[3, 0], torch.tensor([1, e, 1, 1], dtype=F64) / (3 + e + 1))      # exp(0), not scaled, no value
    assert torch.allclose(out[0, 1], torch.tensor([1, 0, 0, 0], dtype=F64) / 6)
    assert abs(float(P.attention(q, k, v, 1.0, lambda i: [i])[2, 0].sum()) - 1.0) < 1e-12


def test_rotation_pairs_halves_and_has_a_magnitude():
    x = torch.zeros(2, 1, 6, dtype=F64)
    x[:, 0, 0], x[:, 0, 5] = 1.0, 7.0
    rot = helpers._scaled_rotation(4, 100.0, (math.e ** 10, 1e9, 1e-3, 1e-4))  # every frequency kept, magnitude 2
    freqs, stretch = P.rotation(rot)
    assert stretch == pytest.approx(2.0) and freqs[0] == 1.0
    got = P.rotate_halves(x, torch.tensor([0, 3]), rot)
    assert torch.allclose(got[0, 0], torch.tensor([2.0, 0, 0, 0, 0, 7.0], dtype=F64))
    assert torch.allclose(got[1, 0], torch.tensor([2 * math.cos(3.0), 0.0, 2 * math.sin(3.0), 0.0, 0.0, 7.0], dtype=F64))


def test_both_sublayers_read_the_same_row(tmp_path):
    """The feed-forward of the plain model sees the norm of the stream ahead of the mixer, and a layer that runs
    another's tensors gives what that layer would give there."""
    config, w = P.read_model(helpers.make_munupel_dir(str(tmp_path), "M1"))
    streams, tokens = [], [5, 9, 200, 17]
    P.forward(config, w, tokens, streams)
    before = w["embed"][tokens]
    for i in (0, 3):
        h = P.layer_norm(before, w["l0.norm1"], w["l0.norm1.b"], 1e-6)
        want = before + P.chunked_attention(h, config["layers"][0]["mixer"], w, "l0.mix.") + P.feed_forward(h, w, "l0.mlp.")
        assert torch.allclose(streams[i], want)
        before = streams[2]
