"""Gararax without a GPU: the configuration's keys and refusals, the running order of repeated layers, what each call keeps
per sequence (kept first pages among them), how heads are laid out, tensor names and shapes, random weights through the
loader, and the plain implementation's own mechanisms against hand-made cases."""
import copy
import os

import numpy as np
import pytest
import torch

import plain_gararax as plain
import tiny_gararax as tiny
from plain_lfm3 import load_folder
from xpu_serve_b200 import registry
from xpu_serve_b200.cache import Cache
from xpu_serve_b200.config import ConfigError, GararaxConfig
from xpu_serve_b200.config.spec import BandRopeScalingSpec, ScaledRopeSpec
from xpu_serve_b200.parts.attention import channel_layout, head_sizes
from xpu_serve_b200.parts.base import KVNeed
from xpu_serve_b200.parts.rope import ScaledRotaryTable
from xpu_serve_b200.weights.expected import expected_tensors
from xpu_serve_b200.weights.loader import load_weights
from xpu_serve_b200.weights.safetensors_io import WeightError, WeightStore, write_safetensors


def test_the_registry_finds_the_design():
    arch = registry.architecture_for(tiny.CONFIGS["A"])
    assert arch.config_class is GararaxConfig
    assert "gararax" in registry.supported_architectures()


@pytest.mark.parametrize("name", sorted(tiny.CONFIGS))
def test_configuration_round_trip(name):
    cfg = GararaxConfig.from_json(tiny.CONFIGS[name])
    assert cfg.to_json() == tiny.CONFIGS[name]
    spec = cfg.model_spec()
    assert len(spec.order) == tiny.layer_runs(name)
    order = plain.running_order(tiny.CONFIGS[name])
    assert [c.layer for c in spec.order] == [i for i, _ in order]
    assert [c.step_row for c in spec.order] == [t for _, t in order]
    assert [c.add_embedding for c in spec.order] == [t is not None and t > 0 for _, t in order]


def test_every_constant_comes_from_the_file():
    spec = GararaxConfig.from_json(tiny.CONFIGS["A"]).model_spec()
    assert spec.tied_head and spec.final_norm.eps == 3e-6 and spec.pass_steps == 2
    l0, l1, l2, l3 = spec.layers
    m = l0.mixer
    assert (m.heads, m.kv_heads, m.head_dim, m.v_dim, m.scale, m.window, m.keep_first) == (6, 3, 12, 20, 0.31, 21, 5)
    assert m.unit_qk and m.qk_norm_eps == 3e-6 and not (m.qkv_bias or m.shared_kv or m.plus_one or m.out_gate or m.head_temp)
    assert m.position == ScaledRopeSpec(12, 100.0, 12, BandRopeScalingSpec(3.0, 1.0, 4.0, 64.0), pairing="interleaved")
    m = l1.mixer
    assert m.shared_kv and m.plus_one and m.out_gate and m.position is None and (m.window, m.keep_first) == (13, 9) and not m.unit_qk
    m = l2.mixer
    assert m.qkv_bias and m.head_temp and m.window == 0 and m.position == ScaledRopeSpec(14, 500.0, 8) and not m.plus_one
    assert (l0.ffn.kind, l0.ffn.intermediate, l0.ffn.eps) == ("poly_norm", 50, 3e-6) and l2.ffn is None
    f = l1.ffn
    assert (f.score, f.experts, f.identity, f.top, f.groups, f.keep_groups, f.group_top, f.renorm) == ("softmax_all", 5, 1, 2, 2, 1, 1, True)
    assert f.shared.intermediate == 12 and not f.shared_gated and f.correction and f.route_scale == 1.0 and l3.ffn.shared is None
    assert all(l.sandwich and l.branch_scale == 0.7 and l.token_side.scale == 0.7 for l in spec.layers)
    assert [l.token_side.offset for l in spec.layers] == [0, 5, 10, 15] and l0.token_side.columns == 20
    c = GararaxConfig.from_json(tiny.CONFIGS["C"]).model_spec()
    assert c.layers[0].token_side is None and c.pass_steps == 0 and not c.adds_embedding
    open_ = copy.deepcopy(tiny.CONFIGS["A"])
    del open_["layers"][0]["mixer"]["mask"]                       # no mask: every earlier position
    del open_["layers"][1]["mixer"]["mask"]["keep_first"]
    o = GararaxConfig.from_json(open_).model_spec()
    assert (o.layers[0].mixer.window, o.layers[0].mixer.keep_first, o.layers[1].mixer.keep_first) == (0, 0, 0)


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
    (("width",), KeyError, "width"), (("norm", "eps"), 0.0, "positive"), (("residual_mult",), KeyError, "residual_mult"),
    (("layers", 0, "type"), "attention_9", "unknown layer type"), (("layers", 0, "mixer", "kv_heads"), 4, "kv_heads"),
    (("layers", 0, "mixer", "rot"), KeyError, "rot"), (("layers", 0, "mixer", "rot", "dims"), 7, "dims"),
    (("layers", 0, "mixer", "rot", "dims"), 14, "dims"), (("layers", 0, "mixer", "rot", "scaling", "high"), 1.0, "scaling"),
    (("layers", 0, "mixer", "mask", "size"), 0, "mask"), (("layers", 0, "mixer", "mask", "keep_first"), -1, "mask"),
    (("layers", 1, "mixer", "vdim"), 12, "vdim"), (("layers", 0, "mixer", "scale"), KeyError, "scale"),
    (("layers", 0, "mlp", "kind"), "gated", "unknown feed-forward"), (("layers", 1, "mlp", "router", "groups", "count"), 4, "groups.count"),
    (("layers", 1, "mlp", "router", "groups", "keep"), 3, "groups.keep"), (("layers", 1, "mlp", "router", "top"), 4, "router.top"),
    (("layers", 1, "mlp", "expert"), KeyError, "expert"), (("layers", 1, "mlp", "shared", "ff"), 0, "positive"),
    (("loop", "stop"), 9, "loop"), (("loop", "times"), 0, "loop"), (("token_side", "dim"), 0, "dim"), (("layers",), [], "layers"),
])
def test_refusals_name_their_key(path, value, word):
    with pytest.raises(ConfigError) as e:
        GararaxConfig.from_json(_broken(path, value))
    assert word in str(e.value)


def test_how_heads_are_laid_out():
    A, B, W = (GararaxConfig.from_json(tiny.CONFIGS[n]).model_spec() for n in ("A", "B", "wide_heads"))
    assert [head_sizes(l.mixer) for l in A.layers] == [(16, 32), (16, 16), (16, 16), (16, 16)]
    assert [head_sizes(l.mixer) for l in B.layers] == [(128, 32), (64, 64), (64, 64), (96, 64)]
    assert [head_sizes(l.mixer) for l in W.layers] == [(160, 128), (48, 136)]
    big = copy.deepcopy(tiny.CONFIGS["B"])                     # both above 32 and at most 64: 64
    big["layers"][1]["mixer"].update(dim=40, vdim=56)
    big["layers"][2]["mixer"].update(dim=36, vdim=36)
    assert [head_sizes(l.mixer) for l in GararaxConfig.from_json(big).model_spec().layers[1:3]] == [(64, 64)] * 2
    # neighbours 2i and 2i + 1 (all twelve channels turn) and halves of the first eight channels go to places i and i + 8
    assert channel_layout(A.layers[0].mixer, 16) == [0, 2, 4, 6, 8, 10, -1, -1, 1, 3, 5, 7, 9, 11, -1, -1]
    assert channel_layout(A.layers[2].mixer, 16) == [0, 1, 2, 3, 8, 9, 10, 11, 4, 5, 6, 7, 12, 13, -1, -1]
    assert channel_layout(A.layers[3].mixer, 16) == list(range(7)) + [-1] * 9
    for spec in (A, B, W):
        for l in spec.layers:
            lay = channel_layout(l.mixer, head_sizes(l.mixer)[0])
            assert sorted(c for c in lay if c >= 0) == list(range(l.mixer.head_dim)) and len(lay) == head_sizes(l.mixer)[0]


def test_what_each_call_keeps():
    """Keys with values of another size, keys alone where they are the values, windows with the first positions; a layer that
    runs twice has two caches of its own."""
    spec = GararaxConfig.from_json(tiny.CONFIGS["A"]).model_spec()
    needs = [registry.arrangement_class(spec.layers[c.layer].kind).cache_need(spec.layers[c.layer]) for c in spec.order]
    assert needs[0] == KVNeed(3, 16, 21, keep_first=5, v_dim=32)
    assert needs[1] == needs[3] == KVNeed(1, 16, 13, planes=1, keep_first=9)
    assert needs[2] == needs[4] == KVNeed(2, 16, 0)
    assert needs[5] == KVNeed(3, 16, 17, planes=1)
    cache = Cache(needs, [None] * 6, 512, dtype=torch.float32, device="cpu")
    assert cache.views[0].storage.shape == (9, 3 * 64 * (16 + 32)) and cache.views[1].storage.shape == (9, 1, 1, 64, 16)
    assert cache.views[1].storage.data_ptr() != cache.views[3].storage.data_ptr()


@pytest.mark.parametrize("window,keep,held_after_400", [(70, 3, {0, 5, 6}), (70, 65, {0, 1, 5, 6}), (70, 0, {5, 6}), (1000, 3, set(range(7)))])
def test_a_window_keeps_the_first_pages(window, keep, held_after_400):
    """Pages behind the window are given back as a sequence grows, the first positions' pages are not; everything goes back at
    the end, and another sequence may then use them."""
    cache = Cache([KVNeed(1, 8, window, keep_first=keep, v_dim=4)], [None], 1024, dtype=torch.float32, device="cpu")
    g = cache.groups[0]
    for grow in ([64] * 6 + [16], [1] * 400, [200, 2, 198], [400]):
        (s,), (other,) = cache.open(1), cache.open(1)
        cache.begin_step([other], [30]); cache.end_step([other], [30])
        done = 0
        for n in grow:
            cache.begin_step([s], [n])
            first = max(0, done - window + 1)
            seen = set(range(first // 64, -(-(done + n) // 64))) | set(range(-(-min(keep, done + n) // 64)))
            assert all(g.table[s, p] >= 0 for p in seen), (done, n)          # what the step's queries can see is held
            cache.end_step([s], [n])
            done += n
            cache.check()
        assert {p for p in range(g.max_seq_pages) if g.table[s, p] >= 0} == held_after_400
        assert cache.tokens_held() == 64 * (len(held_after_400) + 1)
        cache.close([s]); cache.close([other])
        cache.check()
        assert cache.tokens_held() == 0 and (g.table < 0).all()


def test_a_failed_step_leaves_kept_pages_alone():
    cache = Cache([KVNeed(1, 8, 70, keep_first=3)], [None], 1024, dtype=torch.float32, device="cpu")
    (s,) = cache.open(1)
    for n in (300, 100):
        cache.begin_step([s], [n]); cache.end_step([s], [n])
    before = cache.groups[0].table.copy()
    cache.begin_step([s], [120])
    cache.abort_step([s])
    assert (cache.groups[0].table == before).all() and before[s, 0] >= 0
    cache.check()


def test_tensor_names_and_shapes():
    spec = GararaxConfig.from_json(tiny.CONFIGS["A"]).model_spec()
    t = {k: v.shape for k, v in expected_tensors(spec).items()}
    assert t["embed"] == (203, 44) and t["final.norm"] == (44,) and "head" not in t
    assert t["loop.step"] == (2, 44) and t["side.embed"] == (203, 20)
    assert t["l0.mix.q"] == (72, 44) and t["l0.mix.k"] == (36, 44) and t["l0.mix.v"] == (60, 44) and t["l0.mix.o"] == (44, 120)
    assert t["l1.mix.q"] == (40, 44) and t["l1.mix.k"] == (10, 44) and "l1.mix.v" not in t and t["l1.mix.g"] == (40, 44) and t["l1.mix.o"] == (44, 40)
    assert t["l2.mix.q.b"] == (56,) and t["l2.mix.k.b"] == (28,) and t["l2.mix.v.b"] == (12,) and t["l2.mix.temp"] == (4,)
    assert t["l0.mlp.up"] == (50, 44) and t["l0.mlp.down"] == (44, 50) and t["l0.mlp.act"] == (4,) and "l0.mlp.gate" not in t
    assert t["l1.mlp.router"] == (6, 44) and t["l1.mlp.correction"] == (6,) and "l1.mlp.e5.up" not in t
    assert t["l1.mlp.shared.gate"] == (12, 44) and "l1.mlp.shared.sg" not in t and "l3.mlp.shared.gate" not in t
    assert all(t[f"l0.{n}"] == (44,) for n in ("norm1", "norm1b", "norm2", "norm2b")) and "l2.norm2" not in t and "l2.norm2b" not in t
    assert t["l2.side.gate"] == (5, 44) and t["l2.side.proj"] == (44, 5) and t["l2.side.norm"] == (44,)
    c = {k: v.shape for k, v in expected_tensors(GararaxConfig.from_json(tiny.CONFIGS["C"]).model_spec()).items()}
    assert "loop.step" not in c and "side.embed" not in c and not any(".side." in k for k in c)


def test_random_weights_through_the_loader(tmp_path):
    folder = tiny.make_folder(tmp_path, "A", "bfloat16")
    cfg, W = load_folder(folder)
    assert cfg == tiny.CONFIGS["A"]
    spec = GararaxConfig.from_json(cfg).model_spec()
    weights = load_weights(spec, folder)
    assert set(weights) == set(expected_tensors(spec)) and all(weights[f"l2.mix.{n}.b"].abs().min() > 0 for n in "qkv")
    # a missing tensor is named; a layer without a feed-forward may carry the norms of one
    st = WeightStore.open_dir(folder)
    every = {n: st.get(n).clone() for n in st.names()}
    del st
    os.remove(os.path.join(folder, "model.safetensors"))
    write_safetensors(os.path.join(folder, "model.safetensors"), [(n, t) for n, t in every.items() if n != "loop.step"] +
                      [("l2.norm2", every["l1.norm2"]), ("l2.norm2b", every["l1.norm2"]), ("l2.norm3", every["l1.norm2"])])
    with pytest.raises(WeightError) as e:
        load_weights(spec, folder)
    assert "loop.step" in str(e.value) and "l2.norm2" not in str(e.value) and "l2.norm3" in str(e.value)


@pytest.mark.parametrize("scaling", [None, (3.0, 1.0, 4.0, 64), (8.0, 0.5, 2.0, 128), (2.0, 1.0, 1.5, 1000)])
def test_rotation_frequencies_and_table(scaling):
    """The part's frequencies against the oracle's, band by band, and the identity behind the channels that turn."""
    class FakeRuntime:
        shared, device = {}, torch.device("cpu")
    rot = tiny.rotation(12, 100.0, scaling)
    sc = None if scaling is None else BandRopeScalingSpec(*(float(scaling[i]) for i in (0, 1, 2, 3)))
    part = ScaledRotaryTable(ScaledRopeSpec(20, 100.0, 12, sc, pairs=16), FakeRuntime())
    f = plain.frequencies(rot)
    assert np.allclose(part.frequencies()[0].numpy(), f, rtol=1e-12)
    table = part.table(50).double().numpy()
    assert table.shape == (50, 16, 2)
    assert np.abs(table[:, :6, 0] - np.cos(np.arange(50)[:, None] * f)).max() < 1e-7
    assert (table[:, 6:, 0] == 1.0).all() and (table[:, 6:, 1] == 0.0).all()


# --------------------------------------------------------------------------- the plain implementation's own mechanisms
def test_plain_frequencies_by_hand():
    rot = tiny.rotation(4, 100.0)
    assert np.allclose(plain.frequencies(rot), [1.0, 0.1])
    # wavelengths 2 pi and 20 pi; bands: below 10 stays, above 100 is divided by 5, 20 pi lies between
    s = (100.0 / (20 * np.pi) - 1.0) / (10.0 - 1.0)
    got = plain.frequencies(tiny.rotation(4, 100.0, (5.0, 1.0, 10.0, 100)))
    assert np.allclose(got, [1.0, (1 - s) * 0.1 / 5.0 + s * 0.1])
    assert np.allclose(plain.frequencies(tiny.rotation(4, 100.0, (5.0, 1.0, 2.0, 6))), [1.0 / 5.0, 0.1 / 5.0])


def test_plain_rotation_by_hand():
    x = np.zeros((2, 1, 6))
    x[:, 0] = [1.0, 0.0, 0.0, 2.0, 5.0, 7.0]
    r = plain.rotate(x, tiny.rotation(4, 100.0), "interleaved")
    assert np.allclose(r[0], x[0])
    assert np.allclose(r[1, 0], [np.cos(1), np.sin(1), -2 * np.sin(0.1), 2 * np.cos(0.1), 5.0, 7.0])
    r = plain.rotate(x, tiny.rotation(4, 100.0), "half")
    assert np.allclose(r[1, 0], [np.cos(1), -2 * np.sin(0.1), np.sin(1), 2 * np.cos(0.1), 5.0, 7.0])


def test_plain_masks_by_hand():
    see = plain.visible(8, {"size": 3, "keep_first": 2})
    assert list(np.nonzero(see[7])[0]) == [0, 1, 5, 6, 7] and list(np.nonzero(see[3])[0]) == [0, 1, 2, 3] and list(np.nonzero(see[0])[0]) == [0]
    assert list(np.nonzero(plain.visible(5, {"size": 1})[4])[0]) == [4] and plain.visible(4, None)[3].all()


def test_plain_softmax_plus_one_by_hand():
    q, k = np.array([[[1.0]]]), np.array([[[-3.0]]])
    out = plain.softmax_attention(q, k, k, 1.0, np.ones((1, 1), bool), plus_one=True)
    assert np.allclose(out, -3.0 * np.exp(-3.0) / (1.0 + np.exp(-3.0)))
    assert np.allclose(plain.softmax_attention(q, k, k, 1.0, np.ones((1, 1), bool)), -3.0)


def test_plain_poly_norm_by_hand():
    z = np.array([[1.0, -2.0]])
    r1, r2, r3 = np.sqrt(2.5), np.sqrt(8.5), np.sqrt(32.5)
    assert np.allclose(plain.poly_norm(z, np.array([2.0, 3.0, 4.0, 0.5]), 0.0),
                       [[2 / r1 + 3 / r2 + 4 / r3 + 0.5, -4 / r1 + 12 / r2 - 32 / r3 + 0.5]])


def test_plain_routing_by_hand():
    z = np.log(np.array([0.1, 0.2, 0.3, 0.4]))
    ids, w, margin = plain.route(z, np.array([0.5, 0.0, 0.0, 0.0]), 2)
    assert list(ids) == [0, 3] and np.allclose(w, [0.2, 0.8]) and np.isclose(margin, 0.1)     # chosen with the correction, weighted without
    ids, w, margin = plain.route(z, np.array([0.5, 0.0, 0.0, 0.0]), 2, groups=2, keep=1)
    assert list(ids) == [0, 1] and np.allclose(w, [1 / 3, 2 / 3]) and np.isclose(margin, 0.2)  # one group of neighbours stays open
    # closed outputs count as minus infinity: a negative choice score of an open one still wins
    ids, _, _ = plain.route(z, np.array([-5.0, -6.0, -7.0, -7.0]), 2, groups=2, keep=1)
    assert list(ids) == [0, 1]


def test_plain_order_of_looped_layers_and_first_tokens(tmp_path):
    assert plain.running_order(tiny.CONFIGS["B"]) == [(0, None), (1, 0), (1, 1), (1, 2), (2, None), (3, None)]
    assert plain.running_order(tiny.CONFIGS["C"]) == [(0, None), (1, None), (2, None)]
    folder = tiny.make_folder(tmp_path, "whole_loop", "float32")
    cfg, W = load_folder(folder)
    toks = tiny.prompt("whole_loop", 9)
    streams = []
    full = plain.forward(cfg, W, toks, streams)
    assert len(streams) == 6 and np.allclose(full[:4], plain.forward(cfg, W, toks[:4]))       # a prefix does not see what follows
    assert np.allclose(plain.pass_input(np.ones(2), np.array([5.0, 6.0]), 0, np.array([[1.0, 2.0]])), [2.0, 3.0])
    assert np.allclose(plain.pass_input(np.ones(2), np.array([5.0, 6.0]), 1, np.array([[0.0, 0.0], [1.0, 2.0]])), [7.0, 9.0])


def test_the_bench_stacks_are_valid_configurations():
    """`bench.py --workload gararax`: every stack and the stack beside it parse, at equal width and vocabulary."""
    import bench
    for name in bench.GARARAX_STACKS:
        ours, (label, beside) = bench.gararax_stack_configs(name)
        a, b = ours.model_spec(), beside.model_spec()
        assert isinstance(ours, GararaxConfig)
        assert (a.hidden, a.vocab, len(a.layers)) == (b.hidden, b.vocab, len(b.layers)) == (2048, 32768, 2)
