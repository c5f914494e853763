"""Lazovik without a GPU: the configuration's keys and refusals, the running order of repeated layers, what each call keeps per
sequence, how heads are laid out, tensor names and shapes (sizes that the checkpoint decides among them), random weights through
the loader, and the plain implementation's own mechanisms against hand-made cases."""
import copy
import os

import numpy as np
import pytest
import torch

import plain_lazovik as plain
import tiny_lazovik as tiny
from plain_lfm3 import load_folder
from xpu_serve_b200 import registry
from xpu_serve_b200.cache import Cache
from xpu_serve_b200.config import ConfigError, LazovikConfig
from xpu_serve_b200.config.spec import RopeScalingSpec, ScaledRopeSpec
from xpu_serve_b200.parts.attention import head_sizes
from xpu_serve_b200.parts.base import KVNeed, StateNeed
from xpu_serve_b200.parts.rope import ScaledRotaryTable
from xpu_serve_b200.weights.expected import expected_tensors
from xpu_serve_b200.weights.loader import load_weights
from xpu_serve_b200.weights.safetensors_io import WeightError, WeightStore, write_safetensors


def test_the_registry_finds_the_design():
    arch = registry.architecture_for(tiny.CONFIGS["A"])
    assert arch.config_class is LazovikConfig
    assert "lazovik" in registry.supported_architectures()


@pytest.mark.parametrize("name", sorted(tiny.CONFIGS))
def test_configuration_round_trip(name):
    cfg = LazovikConfig.from_json(tiny.CONFIGS[name])
    assert cfg.to_json() == tiny.CONFIGS[name]
    spec = cfg.model_spec()
    assert len(spec.order) == tiny.layer_runs(name)
    order = plain.running_order(tiny.CONFIGS[name])
    assert [c.layer for c in spec.order] == [i for i, _ in order]
    assert [c.step_row for c in spec.order] == [t for _, t in order]
    assert not any(c.add_embedding or c.mix_in for c in spec.order)


def test_every_constant_comes_from_the_file():
    spec = LazovikConfig.from_json(tiny.CONFIGS["A"]).model_spec()
    assert not spec.tied_head and spec.final_norm.eps == 3e-6 and spec.pass_steps == 3 and not any(l.sandwich for l in spec.layers)
    l0, l1, l2, l3 = spec.layers
    a, t = l0.mixer.branches
    assert (a.heads, a.kv_heads, a.head_dim, a.v_dim, a.scale, a.softcap, a.chunk, a.window, a.qkv_taps) == (6, 3, 12, 20, 0.3, 4.0, 13, 0, 2)
    assert a.qk_norm_all and a.qk_norm_eps == 3e-6 and a.qkv_bias and a.o_bias and a.out_gate and not (a.qk_norm or a.unit_qk or a.head_gate)
    assert a.position == ScaledRopeSpec(12, 100.0, 6, RopeScalingSpec(3.0, 64.0, 8.0, 1.0))
    assert (t.heads, t.dim, t.rank, t.eps) == (3, 10, 5, 3e-6) and l0.mixer.scales == (0.8, 1.3) and l2.mixer.scales == (-0.6, 0.7)
    assert l2.mixer.branches[0].position == ScaledRopeSpec(14, 500.0, 14) and l2.mixer.branches[0].qkv_taps == 5
    assert (l1.mixer.heads, l1.mixer.dim, l1.mixer.vdim, l1.mixer.tau, l1.mixer.rank, l1.mixer.eps) == (3, 10, 14, 3.0, 11, 3e-6)
    f = l0.ffn
    assert (f.score, f.activation, f.weight_on, f.experts, f.top, f.intermediate, f.renorm, f.correction) == ("sigmoid", "relu_squared", "input", 6, 2, 20, False, False)
    assert f.shared.intermediate == 12 and f.shared_gated and l1.ffn.shared is None and l2.ffn is None
    open_ = copy.deepcopy(tiny.CONFIGS["A"])
    for key in ("mask", "softcap", "conv"):                       # left out: every earlier position, no cap, no filter
        del open_["layers"][0]["mixer"]["left"][key]
    o = LazovikConfig.from_json(open_).model_spec().layers[0].mixer.branches[0]
    assert (o.chunk, o.softcap, o.qkv_taps) == (0, 0.0, 0)


def _broken(path, value, name="A"):
    cfg = copy.deepcopy(tiny.CONFIGS[name])
    node = cfg
    for key in path[:-1]:
        node = node[key]
    if value is KeyError:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    return cfg


@pytest.mark.parametrize("path,value,word", [
    (("width",), KeyError, "width"), (("norm", "eps"), 0.0, "positive"), (("layers", 0, "type"), "rwkv", "unknown layer type"),
    (("layers", 0, "mixer", "left"), KeyError, "left"), (("layers", 0, "mixer", "right"), KeyError, "right"),
    (("layers", 0, "mixer", "left", "kv_heads"), 4, "kv_heads"), (("layers", 0, "mixer", "left", "rot"), KeyError, "rot"),
    (("layers", 0, "mixer", "left", "rot", "dims"), 7, "dims"), (("layers", 0, "mixer", "left", "rot", "dims"), 14, "dims"),
    (("layers", 0, "mixer", "left", "rot", "scaling", "fast"), 0.0, "scaling"), (("layers", 0, "mixer", "left", "mask", "size"), 0, "mask"),
    (("layers", 0, "mixer", "left", "conv"), 17, "conv"), (("layers", 0, "mixer", "left", "softcap"), -1.0, "softcap"),
    (("layers", 0, "mixer", "left", "scale"), KeyError, "scale"), (("layers", 0, "mixer", "left_scale"), KeyError, "left_scale"),
    (("layers", 0, "mixer", "right", "dim"), 0, "positive"), (("layers", 1, "mixer", "tau"), 0.0, "tau"), (("layers", 1, "mixer", "rank"), 0, "rank"),
    (("layers", 0, "mlp", "kind"), "dense", "unknown feed-forward"), (("layers", 1, "mlp", "router", "top"), 6, "router.top"),
    (("layers", 1, "mlp", "expert"), KeyError, "expert"), (("layers", 0, "mlp", "shared", "ff"), 0, "positive"),
    (("loop", "stop"), 9, "loop"), (("loop", "times"), 0, "loop"), (("layers",), [], "layers"),
])
def test_refusals_name_their_key(path, value, word):
    with pytest.raises(ConfigError) as e:
        LazovikConfig.from_json(_broken(path, value))
    assert word in str(e.value)


def test_what_each_call_keeps():
    """Keys with values of another size, the filters' inputs over all padded channels, the last input, both memories; a layer that
    runs several times has as many caches and states of its own; a filter of one tap keeps nothing."""
    spec = LazovikConfig.from_json(tiny.CONFIGS["A"]).model_spec()
    needs = [registry.arrangement_class(spec.layers[c.layer].kind).cache_need(spec.layers[c.layer]) for c in spec.order]
    a0, a2 = spec.layers[0].mixer.branches[0], spec.layers[2].mixer.branches[0]
    assert head_sizes(a0) == (16, 32) and head_sizes(a2) == (16, 16)
    assert needs[0] == (KVNeed(3, 16, 0, v_dim=32), StateNeed((1, 6 * 16 + 3 * 48), "compute"), StateNeed((44,), "compute"), StateNeed((3, 10, 10), "float32"))
    assert needs[1] == needs[3] == needs[5] == StateNeed((3, 10, 14), "float32")
    assert needs[2] == (KVNeed(1, 16, 0), StateNeed((4, 4 * 16 + 32), "compute"), StateNeed((44,), "compute"), StateNeed((2, 6, 6), "float32"))
    cache = Cache(needs, [None] * len(needs), 512, dtype=torch.float32, device="cpu")
    assert len(cache.views[0]) == 4 and len(cache.views[1]) == 1
    assert len({cache.views[i].storage.data_ptr() for i in (1, 3, 5)}) == 3
    assert len({cache.views[i][3].storage.data_ptr() for i in (0, 2, 4, 6)}) == 4
    c = LazovikConfig.from_json(tiny.CONFIGS["C"]).model_spec().layers[0]
    assert registry.arrangement_class(c.kind).cache_need(c) == (KVNeed(2, 32, 0, v_dim=64), StateNeed((64,), "compute"), StateNeed((1, 24, 24), "float32"))


def test_tensor_names_and_shapes():
    spec = LazovikConfig.from_json(tiny.CONFIGS["A"]).model_spec()
    t = {k: v.shape for k, v in expected_tensors(spec).items()}
    assert t["embed"] == t["head"] == (203, 44) and t["final.norm"] == (44,) and t["loop.step"] == (3, 44)
    p = "l0.mix.left."
    assert t[p + "q"] == (72, 44) and t[p + "k"] == (36, 44) and t[p + "v"] == (60, 44) and t[p + "g"] == (120, 44) and t[p + "o"] == (44, 120)
    assert t[p + "q.b"] == t[p + "q.norm"] == (72,) and t[p + "k.b"] == t[p + "k.norm"] == (36,) and t[p + "v.b"] == (60,) and t[p + "o.b"] == (44,)
    assert t[p + "q.conv"] == (72, 2) and t[p + "k.conv"] == (36, 2) and t[p + "v.conv"] == (60, 2) and p + "v.norm" not in t and p + "g.b" not in t
    p = "l0.mix.right."
    assert all(t[p + f"mu.{s}"] == (44,) for s in "rkvgw") and all(t[p + s] == (30, 44) for s in "rkvg") and t[p + "o"] == (44, 30)
    assert t[p + "w1"] == (5, 44) and t[p + "w2"] == (30, 5) and t[p + "w0"] == t[p + "norm"] == (30,) and t[p + "u"] == (3, 10)
    p = "l1.mix."
    assert t[p + "q"] == t[p + "k"] == (30, 44) and t[p + "v"] == t[p + "g"] == (42, 44) and t[p + "o"] == (44, 42) and t[p + "norm"] == (14,)
    assert t[p + "a1"] == (11, 44) and t[p + "a2"] == (30, 11) and t[p + "a2.b"] == (30,)
    assert t["l0.mlp.router"] == (6, 44) and t["l0.mlp.e5.up"] == (20, 44) and t["l0.mlp.e5.down"] == (44, 20) and "l0.mlp.e0.gate" not in t
    assert t["l0.mlp.shared.up"] == (12, 44) and t["l0.mlp.shared.down"] == (44, 12) and t["l0.mlp.shared.sg"] == (1, 44) and "l1.mlp.shared.up" not in t
    assert t["l0.norm1"] == t["l0.norm2"] == (44,) and "l2.norm2" not in t
    assert "loop.step" not in expected_tensors(LazovikConfig.from_json(tiny.CONFIGS["C"]).model_spec())


def test_sizes_that_the_checkpoint_decides(tmp_path):
    """How many hidden entries a decay has stands in no configuration: a file whose entry names none loads with any number, layer
    by layer, as long as the two matrices of a layer agree; anything else is named."""
    folder = tiny.make_folder(tmp_path, "A", "bfloat16")
    cfg, _ = load_folder(folder)
    for layer in cfg["layers"]:
        layer["mixer"].get("right", layer["mixer"]).pop("rank")
    spec = LazovikConfig.from_json(cfg).model_spec()
    weights = load_weights(spec, folder)
    assert weights["l0.mix.right.w1"].shape == (5, 44) and weights["l1.mix.a2"].shape == (30, 11) and weights["l3.mix.a1"].shape == (7, 44)
    st = WeightStore.open_dir(folder)
    every = {n: st.get(n).clone() for n in st.names()}
    del st
    every["l1.mix.a2"] = every["l1.mix.a2"][:, :9].contiguous()
    every["l2.mix.right.w1"] = every["l2.mix.right.w1"][:, :40].contiguous()
    os.remove(os.path.join(folder, "model.safetensors"))
    write_safetensors(os.path.join(folder, "model.safetensors"), list(every.items()))
    with pytest.raises(WeightError) as e:
        load_weights(spec, folder)
    assert "l1.mix.a2 is [30, 9], expected [30, 11]" in str(e.value) and "l2.mix.right.w1" in str(e.value) and "l0.mix" not in str(e.value)


def test_random_weights_through_the_loader(tmp_path):
    folder = tiny.make_folder(tmp_path, "A", "bfloat16")
    cfg, W = load_folder(folder)
    assert cfg == tiny.CONFIGS["A"]
    spec = LazovikConfig.from_json(cfg).model_spec()
    weights = load_weights(spec, folder)
    assert set(weights) == set(expected_tensors(spec)) and all(weights[f"l0.mix.left.{n}.b"].abs().min() > 0 for n in "qkvo")
    st = WeightStore.open_dir(folder)
    every = {n: st.get(n).clone() for n in st.names()}
    del st
    os.remove(os.path.join(folder, "model.safetensors"))
    write_safetensors(os.path.join(folder, "model.safetensors"), [(n, t) for n, t in every.items() if n != "l0.mix.right.mu.w"] +
                      [("l2.norm2", every["l1.norm2"]), ("l2.norm3", every["l1.norm2"])])
    with pytest.raises(WeightError) as e:
        load_weights(spec, folder)
    assert "l0.mix.right.mu.w" in str(e.value) and "l2.norm2" not in str(e.value) and "l2.norm3" in str(e.value)


@pytest.mark.parametrize("scaling", [None, (3.0, 64, 8.0, 1.0), (8.0, 128, 4.0, 0.5), (2.0, 5000, 32.0, 1.0)])
def test_rotation_frequencies_and_table(scaling):
    """The part's frequencies, factor and table against the oracle's, and the identity behind the channels that turn."""
    class FakeRuntime:
        shared, device = {}, torch.device("cpu")
    rot = tiny.rotation(12, 100.0, scaling)
    sc = None if scaling is None else RopeScalingSpec(*(float(v) for v in scaling))
    part = ScaledRotaryTable(ScaledRopeSpec(20, 100.0, 12, sc, pairs=16), FakeRuntime())
    f, m = plain.frequencies(rot)
    assert np.allclose(part.frequencies()[0].numpy(), f, rtol=1e-12) and np.isclose(part.frequencies()[1], m, rtol=1e-12)
    table = part.table(50).double().numpy()
    assert table.shape == (50, 16, 2)
    assert np.abs(table[:, :6, 0] - m * np.cos(np.arange(50)[:, None] * f)).max() < 2e-7
    assert (table[:, 6:, 0] == 1.0).all() and (table[:, 6:, 1] == 0.0).all()


# --------------------------------------------------------------------------- the plain implementation's own mechanisms
def test_plain_filter_and_mix_by_hand():
    x = np.array([[1.0], [2.0], [4.0]])
    assert np.allclose(plain.causal_filter(x, np.array([[10.0, 1.0]])), [[1.0], [12.0], [24.0]])
    assert np.allclose(plain.causal_filter(x[:1], np.array([[5.0, 10.0, 3.0]])), [[3.0]])
    assert np.allclose(plain.mix_tokens(x, np.array([0.25])), [[0.75], [1.75], [3.5]])


def test_plain_frequencies_by_hand():
    f, m = plain.frequencies(tiny.rotation(4, 100.0))
    assert np.allclose(f, [1.0, 0.1]) and m == 1.0
    # turns over 100 positions: 15.9 and 1.59; index of t turns: 4 ln(100 / (2 pi t)) / (2 ln 100)
    f, m = plain.frequencies(tiny.rotation(4, 100.0, (5.0, 100, 10.0, 1.0)))
    lo, hi = max(np.floor(4 * np.log(100 / (20 * np.pi)) / (2 * np.log(100))), 0), min(np.ceil(4 * np.log(100 / (2 * np.pi)) / (2 * np.log(100))), 3)
    assert (lo, hi) == (0, 2)
    assert np.allclose(f, [1.0, 0.1 / 5 * 0.5 + 0.1 * 0.5]) and np.isclose(m, 0.1 * np.log(5.0) + 1.0)


def test_plain_blocks_and_caps_by_hand():
    see = plain.visible(8, {"size": 3})
    assert list(np.nonzero(see[7])[0]) == [6, 7] and list(np.nonzero(see[5])[0]) == [3, 4, 5] and list(np.nonzero(see[0])[0]) == [0]
    assert list(np.nonzero(plain.visible(5, {"size": 1})[4])[0]) == [4] and plain.visible(4, None)[3].all()
    assert np.allclose(plain.cap_scores(np.array([0.0, 2.0, 1e9]), 2.0), [0.0, 2.0 * np.tanh(1.0), 2.0])


def test_plain_memories_by_hand():
    one = np.ones((2, 1, 1))
    k, v, d = one * np.array([2.0, 3.0])[:, None, None], one * np.array([5.0, 7.0])[:, None, None], one * 0.5
    assert np.allclose(plain.memory(one, k, v, d).ravel(), [10.0, 26.0])                       # 10; 5 + 21
    assert np.allclose(plain.memory_with_bonus(one, k, v, d, np.full((1, 1), 0.1)).ravel(), [1.0, 10.0 + 2.1])     # the second reads the whole first
    assert np.allclose(plain.double_exponential_decay(np.zeros((1, 2)), np.ones((1, 2)), np.ones((1, 1)), np.array([0.0])), np.exp(-1.0))
    assert np.allclose(plain.rooted_sigmoid_decay(np.zeros((1, 2)), np.ones((1, 2)), np.ones((1, 1)), np.array([0.0]), 2.0), np.sqrt(0.5))


def test_plain_routing_by_hand():
    ids, s, margin = plain.route(np.array([0.0, 2.0, -1.0]), 2)
    assert list(ids) == [1, 0] and np.allclose(s, [1 / (1 + np.exp(-2)), 0.5]) and np.isclose(margin, 0.5 - 1 / (1 + np.e))
    w = {"u.up": np.array([[1.0]]), "u.down": np.array([[2.0]])}
    assert np.allclose(plain.weighted_unit(w, "u.", np.array([[3.0]]), 0.5), [[2.0 * 1.5 ** 2]])
    assert np.allclose(plain.weighted_unit(w, "u.", np.array([[3.0]]), 0.5), 0.5 ** 2 * plain.squared_relu_unit(w, "u.", np.array([[3.0]])))


def test_plain_order_of_looped_layers_and_first_tokens(tmp_path):
    assert plain.running_order(tiny.CONFIGS["A"]) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert plain.running_order(tiny.CONFIGS["C"]) == [(0, None), (1, None), (2, None)]
    folder = tiny.make_folder(tmp_path, "whole_loop", "float32")
    cfg, W = load_folder(folder)
    toks = tiny.prompt("whole_loop", 9)
    streams = []
    full = plain.forward(cfg, W, toks, streams)
    assert len(streams) == 6 and np.allclose(full[:4], plain.forward(cfg, W, toks[:4]))       # a prefix does not see what follows
    assert np.allclose(plain.pass_input(np.ones(2), 1, np.array([[0.0, 0.0], [1.0, 2.0]])), [2.0, 3.0])


def test_the_bench_stacks_are_valid_configurations():
    """`bench.py --workload lazovik`: every stack and the stack beside it parse, at equal width and vocabulary."""
    import bench
    for name in bench.LAZOVIK_STACKS:
        ours, (label, beside) = bench.lazovik_stack_configs(name)
        a, b = ours.model_spec(), beside.model_spec()
        assert isinstance(ours, LazovikConfig)
        assert (a.hidden, a.vocab, len(a.layers)) == (b.hidden, b.vocab, len(b.layers)) == (2048, 32768, 2)
