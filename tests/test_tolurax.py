"""The Tolurax decoder without a GPU: configuration, plan, tensor names, cache requests, and the plain
implementation's mechanisms against values worked out by hand."""
import copy
import math

import pytest
import torch

import helpers
import plain_tolurax as P
from llama_rs_metal_b200.config.tolurax import ToluraxConfig
from llama_rs_metal_b200.engine.model import DecoderModel
from llama_rs_metal_b200.errors import InvalidError, UnsupportedError
from llama_rs_metal_b200.parts.base import (CompositeRequest, KeyValueRequest, ModelPlan, ScheduleEntry, StateRequest,
                                            looped_runs)
from llama_rs_metal_b200.parts.linear import GroupedLinear
from llama_rs_metal_b200.parts.rope import RotaryEmbedding
from llama_rs_metal_b200.registry import find_architecture
from llama_rs_metal_b200.runtime import Runtime

F64 = torch.float64


def build(name):
    root = helpers.TOLURAX[name]["config"]
    arch = find_architecture(root)
    config = arch.config_class.from_dict(root)
    return config, arch.plan(config)


def cpu_model(plan):
    return DecoderModel(plan, Runtime(torch.device("cpu"), torch.float32))


# --------------------------------------------------------------------------- configuration and plan
@pytest.mark.parametrize("name", sorted(helpers.TOLURAX))
def test_configuration_reads_every_size_and_writes_it_back(name):
    config, _ = build(name)
    assert ToluraxConfig.from_dict(config.to_dict()) == config
    assert len(config.layers) == len(helpers.TOLURAX[name]["config"]["layers"])


def test_absent_options_are_off():
    config, plan = build("X3")
    assert (config.logit_softcap, config.loops, config.canon_taps) == (None, False, 1)
    assert plan.logit_softcap is None and plan.stream_join is None and not any(e.join_embedding for e in plan.schedule)
    first, last = plan.layers[0].parts["mixer"].params["left"].params, plan.layers[2].parts["mixer"].params["left"].params
    assert first["position"] is None and first["window"] == 1 and last["window"] is None
    assert plan.layers[1].block == "pre_norm_mixer" and plan.layers[0].block == "pre_norm"
    root = copy.deepcopy(helpers.TOLURAX["X3"]["config"])
    del root["canon"]
    bare = cpu_model(find_architecture(root).plan(ToluraxConfig.from_dict(root)))
    assert not any(n.endswith("canon1") for n in bare.tensor_specs())


def test_configuration_names_what_is_missing_or_not_built():
    root = helpers.TOLURAX["X1"]["config"]

    def changed(path, value):
        out = copy.deepcopy(root)
        at = out
        for key in path[:-1]:
            at = at[key]
        if value is None:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        return out
    left = ("layers", 1, "mixer", "left")
    for path, value, word in [(("width",), None, "width"), (("layers", 0, "mixer", "conv"), None, "conv"),
                              (left + ("kv_heads",), 3, "multiple"), (left + ("rot", "dims"), 14, "rot"),
                              (left + ("rot", "scaling", "low"), None, "low"), (left + ("scale",), None, "scale"),
                              (("layers", 3, "mixer", "right", "dim"), 0, "dim"), (("layers", 1, "mixer", "left_scale"), None, "left_scale"),
                              (("canon", "taps"), 0, "taps"), (("logit_softcap",), -1.0, "softcap"), (("loop", "stop"), 9, "loop"),
                              (("norm", "eps"), None, "eps"), (("layers", 0, "mlp", "ff"), None, "ff")]:
        with pytest.raises(InvalidError, match=word):
            ToluraxConfig.from_dict(changed(path, value))
    with pytest.raises(UnsupportedError, match="type"):
        ToluraxConfig.from_dict(changed(("layers", 0, "type"), "delta_2"))
    with pytest.raises(UnsupportedError, match="kind"):
        ToluraxConfig.from_dict(changed(("layers", 0, "mlp", "kind"), "moe"))


def test_the_looped_run_joins_the_embedding_before_every_pass():
    _, plan = build("X1")            # four layers, layers 1 and 2 twice
    assert [(e.layer, e.cache, e.join_embedding) for e in plan.schedule] == [
        (0, 0, False), (1, 1, True), (2, 2, False), (1, 3, True), (2, 4, False), (3, 5, False)]
    assert P.layer_runs(helpers.TOLURAX["X1"]["config"]) == [(e.layer, e.join_embedding) for e in plan.schedule]
    _, plan = build("X2")            # the loop starts at the first layer: the first pass joins too
    assert [e.join_embedding for e in plan.schedule] == [True, False, True, False, True, False, False, False]
    assert looped_runs(3, 1, 1, 5) == [(0, None), (1, None), (2, None)]
    assert looped_runs(3, 1, 2, 3) == [(0, None), (1, 0), (1, 1), (1, 2), (2, None)]


def test_a_schedule_that_joins_needs_a_matrix():
    _, plan = build("X3")
    bad = ModelPlan(**{**plan.__dict__, "schedule": (ScheduleEntry(0, 0, join_embedding=True),)})
    with pytest.raises(InvalidError, match="join"):
        cpu_model(bad)


def test_tensor_names_and_shapes():
    config, plan = build("X1")
    specs = cpu_model(plan).tensor_specs()
    shapes = {name: spec.shape for name, spec in specs.items()}
    assert shapes["embed"] == shapes["head"] == (211, 72) and shapes["loop.in"] == (72, 144)
    assert shapes["final.norm"] == shapes["l0.norm1"] == shapes["l0.norm2"] == (72,) and shapes["l3.canon1"] == (72, 4)
    assert "l1.norm2" not in shapes and "l1.mlp.gate" not in shapes and shapes["l3.mlp.down"] == (72, 40)
    delta = dict(q=(40, 72), k=(40, 72), v=(48, 72), b=(4, 72), a=(4, 72), g=(48, 72), o=(72, 48), A_log=(4,), dt_bias=(4,), norm=(12,))
    delta.update({"q.conv": (40, 2), "k.conv": (40, 2), "v.conv": (48, 2)})
    left = dict(q=(48, 72), k=(24, 72), v=(40, 72), g=(80, 72), o=(72, 80), pb=(4,))
    left.update({"q.norm": (12,), "k.norm": (12,)})
    right = dict(r=(30, 72), k=(30, 72), v=(30, 72), g=(30, 72), o=(72, 30), w1=(5, 72), w2=(30, 5), w0=(30,), u=(3, 10), norm=(30,))
    right.update({"mu." + s: (72,) for s in "rkvgw"})
    for prefix, own in (("l0.mix.", delta), ("l1.mix.left.", left), ("l1.mix.right.", right)):
        for name, shape in own.items():
            assert shapes[prefix + name] == shape, prefix + name
        assert len([n for n in shapes if n.startswith(prefix)]) == len(own)
    root = copy.deepcopy(helpers.TOLURAX["X1"]["config"])      # without decay_rank the rank is the checkpoint's
    del root["layers"][1]["mixer"]["right"]["decay_rank"]
    open_specs = cpu_model(find_architecture(root).plan(ToluraxConfig.from_dict(root))).tensor_specs()
    assert open_specs["l1.mix.right.w1"].shape == (None, 72) and open_specs["l1.mix.right.w2"].fits((30, 9))


def test_cache_requests_keep_what_each_layer_needs():
    _, plan = build("X1")
    requests = cpu_model(plan).cache_requests()
    canon = StateRequest((3, 72), torch.float32)
    assert requests[0] == CompositeRequest((CompositeRequest((StateRequest((4, 20, 12)), StateRequest((1, 128)))), canon))
    time_mix = CompositeRequest((StateRequest((3, 10, 10)), StateRequest((1, 72))))
    assert requests[1] == requests[3] == CompositeRequest((CompositeRequest((KeyValueRequest(2, 12, 7, 20), time_mix)), canon))
    _, plan = build("X3")            # one tap in both convolutions: no tails
    requests = cpu_model(plan).cache_requests()
    assert requests[1] == StateRequest((1, 8, 8)) and isinstance(requests[0].parts[0], KeyValueRequest)


def test_stretched_frequencies_agree_with_the_position_encoding():
    for rot in (helpers._rotation(32, 10000.0, (4.0, 1.0, 2.0, 100.0)), helpers._rotation(80, 30000.0, (6.0, 1.5, 5.0, 512.0)),
                helpers._rotation(6, 50.0)):
        s = rot.get("scaling")
        params = dict(scaling="llama3", factor=s["factor"], low_freq_factor=s["low"], high_freq_factor=s["high"],
                      original_max_position_embeddings=int(s["original"])) if s else {}
        ours = torch.tensor(RotaryEmbedding(128, rot["dims"], rot["base"], **params).inverse_frequencies(), dtype=F64)
        assert torch.allclose(ours, P.frequencies(rot), rtol=1e-12)
        if s:                        # each of the three cases occurs
            plain = P.frequencies(dict(rot, scaling=None))
            ratio = P.frequencies(rot) / plain
            assert (ratio == 1).any() and (ratio * s["factor"] - 1).abs().min() < 1e-12 and ((ratio < 1) & (ratio * s["factor"] > 1 + 1e-9)).any()


def test_attention_options_that_exclude_each_other():
    from llama_rs_metal_b200.parts.attention import Attention
    with pytest.raises(InvalidError, match="gate"):
        Attention(64, 2, 1, 16, gate="head", weights="sigmoid")
    with pytest.raises(UnsupportedError, match="weights"):
        Attention(64, 2, 1, 16, weights="relu")
    assert Attention(64, 2, 1, 16).mixed_width is None
    assert Attention(64, 2, 1, 16, value_dim=24, weights="sigmoid").mixed_width == 48


def test_grouped_matrices_are_filled_up_to_whole_tiles():
    mats = [torch.full((n, 8), float(i + 1)) for i, n in enumerate((30, 200, 5))]
    g = GroupedLinear(mats)
    assert g.group_cols == 256 and tuple(g.weight.shape) == (517, 8)
    for i, m in enumerate(mats):
        rows = g.weight[g.column(i):g.column(i) + m.shape[0]]
        assert torch.equal(rows, m)
    assert float(g.weight.sum()) == sum(float(m.sum()) for m in mats)


# --------------------------------------------------------------------------- the plain mechanisms by hand
def test_norm_convolution_and_softcap_by_hand():
    x = torch.tensor([[1.0, 3.0]], dtype=F64)
    assert torch.allclose(P.layer_norm(x, torch.tensor([2.0, 5.0], dtype=F64), 0.0), torch.tensor([[-2.0, 5.0]], dtype=F64))
    assert torch.allclose(P.layer_norm(x, torch.ones(2, dtype=F64), 3.0), torch.tensor([[-0.5, 0.5]], dtype=F64))   # eps inside the root
    u = torch.tensor([[1.0], [2.0], [3.0], [4.0]], dtype=F64)
    taps = torch.tensor([[100.0, 10.0, 1.0]], dtype=F64)     # the last tap is the current token's
    assert torch.equal(P.causal_conv(u, taps), torch.tensor([[1.0], [12.0], [123.0], [234.0]], dtype=F64))
    z = torch.tensor([1.0, 100.0], dtype=F64)
    assert torch.allclose(P.softcap(z, 2.0), torch.tensor([2.0 * math.tanh(0.5), 2.0], dtype=F64))
    assert torch.equal(P.softcap(z, None), z)


def test_sigmoid_weights_are_not_normalized_and_end_with_the_window():
    T = 6
    q, k = torch.ones(T, 2, 1, dtype=F64), torch.zeros(T, 1, 1, dtype=F64)
    k[1] = 5.0
    v = torch.eye(T, dtype=F64).reshape(T, 1, T)
    out = P.sigmoid_attention(q, k, v, 0.5, torch.tensor([0.0, -1.0], dtype=F64), 3).reshape(T, 2, T)
    far, mid = 1.0 / (1.0 + math.exp(-2.5)), 0.5
    assert torch.allclose(out[3, 0], torch.tensor([0, far, mid, mid, 0, 0], dtype=F64))        # itself and two before
    assert torch.allclose(out[4, 0], torch.tensor([0, 0, mid, mid, mid, 0], dtype=F64))
    assert torch.allclose(out[0, 0], torch.tensor([mid, 0, 0, 0, 0, 0], dtype=F64))
    assert abs(float(out[3, 1, 1]) - 1.0 / (1.0 + math.exp(-1.5))) < 1e-12                     # the second head's offset
    everything = P.sigmoid_attention(q, k, v, 0.5, torch.zeros(2, dtype=F64), None).reshape(T, 2, T)
    assert float(everything[5, 0, 0]) == 0.5


def test_delta_and_bonus_recurrences_with_one_channel():
    gen = torch.Generator().manual_seed(4)
    q, k, v = (torch.randn(5, 1, 1, generator=gen, dtype=F64) for _ in range(3))
    g, b = torch.rand(5, 1, generator=gen, dtype=F64), torch.rand(5, 1, generator=gen, dtype=F64)
    S, want = 0.0, []
    for t in range(5):
        S = float(g[t]) * S
        S += float(k[t]) * float(b[t]) * (float(v[t]) - S * float(k[t]))
        want.append(S * float(q[t]))
    assert torch.allclose(P.delta_scan(q, k, v, g, b).reshape(-1), torch.tensor(want, dtype=F64))
    bonus, S, want = 0.7, 0.0, []
    for t in range(5):
        kv = float(k[t]) * float(v[t])
        want.append((S + bonus * kv) * float(q[t]))          # read before the write
        S = float(g[t]) * S + kv
    got = P.bonus_scan(q, k, v, g.reshape(5, 1, 1), torch.tensor([[bonus]], dtype=F64))
    assert torch.allclose(got.reshape(-1), torch.tensor(want, dtype=F64))


def test_rotation_pairs_halves():
    x = torch.zeros(2, 1, 6, dtype=F64)
    x[:, 0, 0], x[:, 0, 5] = 1.0, 7.0
    got = P.rotate_halves(x, torch.tensor([0, 3]), helpers._rotation(4, 100.0))
    assert torch.equal(got[0], x[0])
    assert torch.allclose(got[1, 0], torch.tensor([math.cos(3.0), 0.0, math.sin(3.0), 0.0, 0.0, 7.0], dtype=F64))


def test_the_loop_replaces_the_stream_before_each_pass(tmp_path):
    """A model whose sublayers add nothing: the stream is W [x; x0] applied once per pass."""
    def silence(tensors):
        for name, t in tensors.items():
            if name.endswith((".o", ".down")):
                t.zero_()
    config, w = P.read_model(helpers.make_tolurax_dir(str(tmp_path), "X2", edit=silence))
    streams, tokens = [], [5, 9, 200]
    P.forward(config, w, tokens, streams)
    x0 = w["embed"][tokens]
    x = x0
    for t in range(3):
        x = torch.cat([x, x0], dim=1) @ w["loop.in"].T
        assert torch.allclose(streams[2 * t], x) and torch.allclose(streams[2 * t + 1], x)
    assert torch.allclose(streams[-1], x)
