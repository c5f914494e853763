"""Gararax on the device against the plain float64 implementation (plain_gararax.py): single-mechanism models, the replay
schedules (whole; the last tokens one by one; unequal batches one after another, so that slots and pages are used again;
prompts in pieces down to two tokens beside single tokens), long decoding across page borders and past kept pages, first
tokens, keys just inside and outside windows and kept positions (planted, at the kernels and through the model), the kernels
of each mechanism alone, planted mistakes, greedy generation through the engine and the command line."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_gararax as plain
import tiny_gararax as tiny
import trace_util as tu
from plain_lfm3 import load_folder

pytestmark = pytest.mark.gpu

COS = {"float32": 0.999999, "bfloat16": 0.97}
LENGTHS = [1, 2, 7, 16, 23, 40, 70, 5, 13, 33, 64, 65, 131]
CLOSE_CALL = {"float32": 1e-5, "bfloat16": 0.008}


def requests_for(name, lengths=LENGTHS):
    return {f"r{i}": tiny.prompt(name, n, salt=i) for i, n in enumerate(lengths)}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("gararax_models")
    made = {}

    def get(name, dtype):
        if (name, dtype) not in made:
            made[(name, dtype)] = tiny.make_folder(root, name, dtype)
        return made[(name, dtype)]
    return get


@pytest.fixture(scope="module")
def replayers(folders):
    from xpu_serve_b200.engine.model import load_model
    from xpu_serve_b200.engine.replay import Replayer
    made = {}

    def get(name, dtype, max_tokens=1024):
        key = (name, dtype, max_tokens)
        if key not in made:
            made[key] = Replayer(load_model(folders(name, dtype), dtype=dtype), max_tokens, None)
        return made[key]
    return get


_REFS = {}


def reference(folder, requests, dtype="float32"):
    """{(request, position): float64 logits}, memoised per folder and request. A token whose choice of units is a close call
    at this precision may choose otherwise on the device, and every later position of its sequence may see that (through the
    keys and values): those are left out."""
    cfg, W = load_folder(folder)
    out = {}
    for rid, toks in requests.items():
        key = (folder, tuple(toks))
        if key not in _REFS:
            margins: list = []
            logits = plain.forward(cfg, W, toks, margins=margins)
            _REFS[key] = (logits, np.min(np.stack(margins), 0) if margins else np.full(len(toks), np.inf))
        logits, margins = _REFS[key]
        close = np.nonzero(margins < CLOSE_CALL[dtype])[0]
        for p in range(len(toks) if close.size == 0 else int(close[0])):
            out[(rid, p)] = logits[p]
    return out


def check(name, dtype, steps, requests, replayers, folders, max_tokens=1024, replayer=None, least=8, ref=None):
    rp = replayer or replayers(name, dtype, max_tokens)
    got = tu.collect(steps, tu.run_in_process(rp, steps), tiny.CONFIGS[name]["vocab"])
    ref = reference(folders(name, dtype), requests, dtype) if ref is None else ref
    ref = {k: v for k, v in ref.items() if k in got}
    assert len(ref) >= min(len(got), least), "the test's first tokens are close calls of a router; pick other prompts"
    gap, where, cos = tu.worst_gap({k: v for k, v in got.items() if k in ref}, ref)
    tol = tiny.upper_limit(name, dtype)
    print(f"GAP gararax {name} {dtype} steps={len(steps)} places={len(ref)} of {len(got)} gap={gap:.3e} at {where} cos={cos:.7f} tol={tol:.1e}")
    assert gap <= tol, f"{name} {dtype}: gap {gap:.3e} at {where}"
    assert cos >= COS[dtype], f"{name} {dtype}: cosine {cos}"
    rp.cache.check()
    assert rp.cache.slots.held_count == 0 and rp.cache.tokens_held() == 0
    return got


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["normed", "shared_values", "tempered", "poly", "routed", "whole_loop", "wide_heads"])
def test_one_mechanism_alone(name, dtype, replayers, folders):
    """Models of one layer (the one whose every layer repeats, and one whose heads only the generic kernels take, beside them):
    whole prompts (a sequence of one and of two tokens among them), the tail token by token, unequal requests together."""
    reqs = requests_for(name, [1, 2, 11, 37, 90])
    check(name, dtype, tu.whole_trace(reqs), reqs, replayers, folders)
    check(name, dtype, tu.tail_trace(reqs, tail=20), reqs, replayers, folders)
    check(name, dtype, tu.batch_trace(reqs, 3), reqs, replayers, folders)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_whole(name, dtype, replayers, folders):
    reqs = requests_for(name)
    check(name, dtype, tu.whole_trace(reqs), reqs, replayers, folders)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_prefill_then_token_by_token(name, dtype, replayers, folders):
    reqs = requests_for(name)
    check(name, dtype, tu.tail_trace(reqs, tail=32), reqs, replayers, folders)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("batch", [3, 5, 13])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_unequal_batches_one_after_another(name, batch, dtype, replayers, folders):
    """Batches of unequal requests against each alone; a later batch takes the slots and pages that the one before gave back,
    in a cache that holds little more than one batch."""
    reqs = requests_for(name)
    check(name, dtype, tu.batch_trace(reqs, batch), reqs, replayers, folders, max_tokens=1280)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("pieces", [(2, 3, 64, 5), (7, 64, 65, 129, 3, 16, 40), (130, 2)])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_prompts_in_pieces(name, pieces, dtype, replayers, folders):
    """Pieces of several sizes, down to two tokens, at page borders, in steps that mix a later piece of one request with
    single tokens of others: a piece's first tokens find the window's keys and the kept ones, every pass over the repeated
    layers its own."""
    reqs = requests_for(name, [131, 2, 70, 23, 140, 64, 9])
    check(name, dtype, tu.pieces_trace(reqs, 4, pieces=pieces), reqs, replayers, folders)


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "float32"), ("C", "float32"), ("D", "bfloat16"), ("whole_loop", "bfloat16"),
                                        ("normed", "bfloat16"), ("shared_values", "bfloat16")])
def test_long_decoding(name, dtype, replayers, folders):
    """A short prompt and 260 tokens one by one: four page borders are crossed, pages fall out of the windows and are given
    back while the kept ones stay; beside it a second request that ends early."""
    reqs = {"long": tiny.prompt(name, 264, salt=3), "short": tiny.prompt(name, 30, salt=4)}
    check(name, dtype, tu.batch_trace(reqs, 2, prompt_frac=0.02), reqs, replayers, folders)


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "float32"), ("D", "float32"), ("D", "bfloat16")])
def test_long_prompts(name, dtype, replayers, folders):
    """Prompts of 306 and 446 tokens beside one of 46 in one step (more than one attention tile each, windows that skip whole
    pages between the kept positions and their own), then single tokens."""
    reqs = {"a": tiny.prompt(name, 306, salt=5), "b": tiny.prompt(name, 446, salt=6), "c": tiny.prompt(name, 46, salt=7)}
    check(name, dtype, tu.batch_trace(reqs, 3, prompt_frac=0.985), reqs, replayers, folders, max_tokens=1280, least=4)


def test_pages_used_again_hold_nothing_over(folders):
    """The whole cache is filled with large numbers before and between batches: what a step reads it has written itself."""
    from xpu_serve_b200.engine.model import load_model
    from xpu_serve_b200.engine.replay import Replayer
    for name, dtype in (("B", "bfloat16"), ("A", "float32")):
        reqs = requests_for(name, [70, 131, 5, 64])
        ref = reference(folders(name, dtype), reqs, dtype)
        rp = Replayer(load_model(folders(name, dtype), dtype=dtype), 640, None)
        for value in (float("nan"), 1e4):
            for g in rp.cache.groups:
                for t in g.storage.values():
                    t.fill_(value)
            check(name, dtype, tu.batch_trace(reqs, 4), reqs, None, folders, replayer=rp, ref=ref)


# -------------------------------------------------------------------------- windows, kept positions, far keys in a model
def edge_model(kind, size, keep):
    """A one-layer model with sharp scores, so that a single key decides most of a softmax."""
    if kind == "normed":
        layer = tiny.normed(4, 2, 16, 32, 1.5, tiny.rotation(8, 100.0), size, keep)
    else:
        layer = tiny.shared(4, 2, 32, 1.2, size, keep)
    return tiny.model(64, 120, [(layer, None)], mult=1.0)


def sees(cfg, W, toks, positions, change):
    """Largest change of the logits at each position, relative to the largest logit, when the oracle's mask is changed."""
    other = copy.deepcopy(cfg)
    other["layers"][0]["mixer"]["mask"].update(change)
    a, b = plain.forward(cfg, W, toks), plain.forward(other, W, toks)
    return np.abs(a - b)[positions].max(-1) / np.abs(a).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["normed", "shared"])
@pytest.mark.parametrize("size,keep", [(64, 6), (37, 64), (100, 1), (20, 90)])
def test_a_key_at_an_edge_through_the_model(kind, size, keep, dtype, tmp_path):
    """One attention layer with sharp scores; the oracle with a window one position longer or shorter, or one more or one fewer
    position kept, moves by far more than the bound at several positions, in the prompt's part and in the decoded part, so the
    model's agreement with the oracle is agreement about the edges: whole, the last 70 tokens one by one, in pieces."""
    from xpu_serve_b200.config import GararaxConfig
    from xpu_serve_b200.engine.model import load_model
    from xpu_serve_b200.engine.replay import Replayer
    from xpu_serve_b200.weights import write_random_model
    cfg = edge_model(kind, size, keep)
    folder = str(tmp_path / "sharp")
    write_random_model(folder, GararaxConfig.from_json(cfg), seed=5, dtype=dtype, std=0.15, norm_range=(0.5, 1.5), scale={"embed": 6.0})
    _, W = load_folder(folder)
    toks = [int(t) for t in np.random.default_rng(size + keep).integers(0, 120, 220)]
    tol = 2e-5 if dtype == "float32" else 1.5e-2
    for change in ({"size": size + 1}, {"size": size - 1}, {"keep_first": keep + 1}, {"keep_first": keep - 1}):
        moved = sees(cfg, W, toks, np.arange(100, 220), change)
        if dtype == "float32":
            for part in (moved[:50], moved[50:]):
                assert (part > 20 * tol).sum() >= 2, (change, np.sort(part)[-3:])
        else:
            assert moved.max() > 2 * tol, (change, np.sort(moved)[-3:])
    ref = plain.forward(cfg, W, toks)
    reqs = {"far": toks, "near": toks[50:116]}
    rp = Replayer(load_model(folder, dtype=dtype), 1024, None)
    for steps in (tu.whole_trace(reqs), tu.tail_trace(reqs, tail=70), tu.pieces_trace(reqs, 2, pieces=(63, 2, 64, 5)), tu.batch_trace(reqs, 2)):
        got = tu.collect(steps, tu.run_in_process(rp, steps), 120)
        want = {("far", p): ref[p] for p in range(220)}
        gap, where, cos = tu.worst_gap({k: got[k] for k in want}, want)
        assert gap <= tol, (len(steps), gap, where)
    assert rp.cache.slots.held_count == 0


def test_far_keys_through_the_model(tmp_path):
    """Attention over every earlier position, sharp: the last positions of a 200-token prompt hang on the first page's tokens."""
    from xpu_serve_b200.config import GararaxConfig
    from xpu_serve_b200.engine.model import load_model
    from xpu_serve_b200.engine.replay import Replayer
    from xpu_serve_b200.weights import write_random_model
    cfg = tiny.model(64, 150, [(tiny.tempered(4, 2, 32, 16, 3.0, tiny.rotation(8, 50.0)), None)], mult=1.0)
    folder = str(tmp_path / "sharp")
    write_random_model(folder, GararaxConfig.from_json(cfg), seed=5, dtype="float32", std=0.15, norm_range=(0.5, 1.5), scale={"embed": 6.0})
    _, W = load_folder(folder)
    toks = [int(t) for t in np.random.default_rng(1).integers(0, 150, 200)]
    ref = plain.forward(cfg, W, toks)
    other = plain.forward(cfg, W, [(t + 7) % 150 for t in toks[:64]] + toks[64:])
    moved = np.abs(ref[150:] - other[150:]).max() / np.abs(ref).max()
    tol = 2e-5
    assert moved > 20 * tol, f"the far keys do not matter here ({moved:.2e})"
    reqs = {"far": toks}
    rp = Replayer(load_model(folder, dtype="float32"), 1024, None)
    for steps in (tu.whole_trace(reqs), tu.tail_trace(reqs, tail=70), tu.pieces_trace(reqs, 1, pieces=(63, 2, 64, 5))):
        got = tu.collect(steps, tu.run_in_process(rp, steps), 150)
        gap, where, _ = tu.worst_gap(got, {("far", p): ref[p] for p in range(200)})
        assert gap <= tol, (len(steps), gap, where)


# ------------------------------------------------------------------------------------------------ planted mistakes
MISTAKES = {
    "the side input left out": lambda m: m.setattr(plain, "token_side", lambda cfg, w, i, tokens, s: 0.0),
    "a pass without the embedding": lambda m: m.setattr(plain, "pass_input", lambda s, s0, t, step: s + step[t]),
    "a pass without its vector": lambda m: m.setattr(plain, "pass_input", lambda s, s0, t, step: s + s0 if t else s),
    "no one in the denominator": lambda m: m.setattr(
        plain, "softmax_attention", lambda *a, _f=plain.softmax_attention, plus_one=False: _f(*a)),
    "the other pairing": lambda m: m.setattr(
        plain, "rotate", lambda x, rot, pairing, *a, _f=plain.rotate: _f(x, rot, {"half": "interleaved", "interleaved": "half"}[pairing], *a)),
    "no frequency scaling": lambda m: m.setattr(plain, "frequencies", lambda rot, _f=plain.frequencies: _f({**rot, "scaling": None})),
    "no groups": lambda m: m.setattr(plain, "route", lambda z, c, top, groups=1, keep=1, _f=plain.route: _f(z, c, top)),
    "no correction": lambda m: m.setattr(plain, "choice_scores", lambda z, c, _f=plain.choice_scores: _f(z, 0.0 * c)),
    "no constant in the cubic": lambda m: m.setattr(
        plain, "poly_norm", lambda z, act, eps, _f=plain.poly_norm: _f(z, np.array([*act[:3], 0.0]), eps)),
    "a window one longer": lambda m: m.setattr(
        plain, "visible", lambda T, mask, _f=plain.visible: _f(T, {**mask, "size": mask["size"] + 1} if mask else None)),
    "one kept position fewer": lambda m: m.setattr(
        plain, "visible", lambda T, mask, _f=plain.visible: _f(T, {**mask, "keep_first": mask["keep_first"] - 1} if mask else None)),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_a_mistake_leaves_the_bounds(mistake, replayers, folders, monkeypatch):
    """What the device gives for model A against an oracle with one mistake in it: outside the bound."""
    reqs = requests_for("A", [40, 70])
    steps = tu.tail_trace(reqs, tail=10)
    check("A", "float32", steps, reqs, replayers, folders)
    cfg, W = load_folder(folders("A", "float32"))
    MISTAKES[mistake](monkeypatch)
    wrong = {(r, p): l for r, toks in reqs.items() for p, l in enumerate(plain.forward(cfg, W, toks))}
    monkeypatch.undo()
    with pytest.raises(AssertionError, match="gap"):
        check("A", "float32", steps, reqs, replayers, folders, ref=wrong)


# ------------------------------------------------------------------------------------------------- the kernels alone
def dev_i32(v):
    return torch.tensor(np.asarray(v), dtype=torch.int32, device="cuda")


ATTENTION_SHAPES = [   # H, G, D, DV, planes
    (4, 2, 64, 64, 2), (4, 2, 64, 64, 1), (8, 2, 128, 32, 2), (4, 4, 48, 128, 2), (3, 1, 96, 64, 2), (6, 2, 16, 32, 2), (2, 2, 32, 32, 1),
    (20, 1, 64, 32, 2), (2, 1, 160, 72, 2), (2, 1, 128, 128, 1)]


@pytest.mark.parametrize("kernel", ["generic f32", "generic", "mma", "mma split", "decode", "decode split", "decode merged", "tcgen05"])
@pytest.mark.parametrize("shape", ATTENTION_SHAPES, ids=str)
@pytest.mark.parametrize("window,keep,plus_one,gated", [(0, 0, True, "channels"), (40, 5, False, None), (64, 64, True, "channels"),
                                                        (100, 70, True, "heads"), (1, 1, False, None), (17, 0, False, "channels")])
def test_attention_kernels(kernel, shape, window, keep, plus_one, gated):
    """Queries of several sequences in one launch, pages in a shuffled order, pages that no query can see given back (their
    numbers are -1) and every unwritten place of the cache a NaN. For the last query of two sequences the keys on both sides
    of the window's edge and of the kept positions' edge, at page borders, far back and at the query itself point along the
    query, so that leaving one out or letting one in changes the result by far more than the bound."""
    from xpu_serve_b200.ops import lib as ops
    H, G, D, DV, planes = shape
    dtype = torch.float32 if kernel == "generic f32" else torch.bfloat16
    decode = kernel.startswith("decode")
    if kernel == "tcgen05" and not (D == DV and ops.attention_tc_supports(D, 64, H // G)):
        pytest.skip("the tcgen05 kernel does not take this shape")
    if not kernel.startswith("generic") and kernel != "tcgen05" and not ops.attention_mma_supports(D, 64, H // G, DV):
        pytest.skip("the tensor-core kernels do not take this shape")
    if decode and H // G > 16 and "merged" in kernel:
        pytest.skip("merging inside the kernel takes groups of at most 16")
    torch.manual_seed(11)
    page, scale = 64, 0.9
    lens = [300, 129, 64, 1]
    q_lens = [1, 1, 1, 1] if decode else [140, 70, 9, 1] if kernel == "tcgen05" else [33, 5, 2, 1]
    n_pages = sum(-(-n // page) for n in lens)
    order = torch.randperm(n_pages + 3)
    page_shape = ops.kv_page_shape(G, page, D, DV, planes)
    pool = torch.full((n_pages + 4, *page_shape), float("nan"), dtype=dtype)
    flat = pool.view(n_pages + 4, -1)
    k_view = flat[:, :G * page * D].view(-1, G, page, D)
    v_view = k_view if planes == 1 else flat[:, G * page * D:].view(-1, G, page, DV)
    keys = [torch.randn(n, G, D) * 0.3 for n in lens]
    values = [torch.randn(n, G, DV) for n in lens]
    T = sum(q_lens)
    q = torch.randn(T, H, D) * 0.3
    positions = [p for n, ql in zip(lens, q_lens) for p in range(n - ql, n)]
    seq_of = [s for s, ql in enumerate(q_lens) for _ in range(ql)]
    ends = np.cumsum(q_lens)
    mask = {"size": window, "keep_first": keep} if window else None
    see_all = [plain.visible(n, mask) for n in lens]
    for s in (0, 1):
        t, pos = int(ends[s]) - 1, lens[s] - 1
        for j in {3, 63, 64, pos - window + 1, pos - window, keep - 1, keep, pos}:
            if 0 <= j <= pos:
                keys[s][j, 0] = q[t, 0] / q[t, 0].norm() * 3.0 + torch.randn(D) * 0.3
    table = torch.full((len(lens), 5), -1, dtype=torch.int32)
    at = 0
    for s, n in enumerate(lens):
        k = keys[s].to(dtype)
        v = k if planes == 1 else values[s].to(dtype)
        keys[s], values[s] = k.double().numpy(), v.double().numpy()
        seen = see_all[s][n - q_lens[s]:].any(0)
        for p in range(-(-n // page)):
            if not seen[p * page:(p + 1) * page].any():
                continue
            table[s, p] = int(order[at]); at += 1
            m = min(page, n - p * page)
            k_view[int(table[s, p]), :, :m] = k[p * page:p * page + m].transpose(0, 1)
            v_view[int(table[s, p]), :, :m] = v[p * page:p * page + m].transpose(0, 1)
    pool, qd = pool.cuda(), q.to(dtype).cuda()
    gate = None
    columns = H * DV if gated == "channels" else H
    if gated:
        wide = torch.randn(T, columns + 16).to(dtype).cuda()
        gate = wide[:, 8:8 + columns]
    opts = dict(keep=keep, planes=planes, plus_one=plus_one, gate_channels=gated == "channels")
    out = torch.full((T, H, DV), float("nan"), dtype=dtype, device="cuda")
    cu = dev_i32([0] + list(ends))
    if kernel.startswith("generic"):
        ops.attention_generic(qd, pool, table.cuda(), dev_i32(seq_of), dev_i32(positions), gate, out, G, page, scale, window, **opts)
    elif kernel == "tcgen05":
        ops.attention_tc(qd, pool, table.cuda(), cu, dev_i32(lens), gate, out, len(lens), max(q_lens), G, page, scale, window, max(lens), **opts)
    else:
        splits = 3 if "split" in kernel or "merged" in kernel else 1
        scratch = torch.empty(ops.attention_mma_scratch_bytes(T * H, DV, splits) + 16, dtype=torch.uint8, device="cuda") if splits > 1 else None
        counters = torch.zeros(len(lens) * G, dtype=torch.int32, device="cuda") if "merged" in kernel else None
        ops.attention_mma(qd, pool, table.cuda(), cu, dev_i32(lens), gate, out, scratch, len(lens), max(q_lens), G, page, scale,
                          window, splits, counters=counters, bounded_waits=decode, **opts)
        assert counters is None or int(counters.abs().sum()) == 0
    assert int(ops.gemm_tc_status("cuda").item()) == 0
    got = out.double().cpu().numpy()
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    rows = qd.double().cpu().numpy()

    def oracle(s, see):
        n, ql = lens[s], q_lens[s]
        full = np.zeros((n, H, D))
        full[n - ql:] = rows[int(ends[s]) - ql:int(ends[s])]
        o = plain.softmax_attention(full, keys[s], values[s], scale, see, plus_one=plus_one)[n - ql:]
        if gated:
            g = plain.sigmoid(gate[int(ends[s]) - ql:int(ends[s])].double().cpu().numpy())
            o = o * (g.reshape(ql, H, DV) if gated == "channels" else g[:, :, None])
        return o

    changes = ({"size": window + 1, "keep_first": keep}, {"size": window - 1, "keep_first": keep}, {"size": window, "keep_first": keep + 1})
    moved = np.zeros(len(changes))
    for s in range(len(lens)):
        want = oracle(s, see_all[s])
        have = got[int(ends[s]) - q_lens[s]:int(ends[s])]
        scale_of = max(np.abs(want).max(), 1e-3)
        assert np.abs(have - want).max() / scale_of < tol, (kernel, s)
        if s < 2 and 1 < window <= 64:
            moved = np.maximum(moved, [np.abs(oracle(s, plain.visible(lens[s], c))[-1] - want[-1]).max() / scale_of for c in changes])
    if 1 < window <= 64:                      # the planted keys make the edges show
        assert (moved > 2 * tol).all(), moved


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,DV,planes", [(4, 2, 16, 32, 2), (8, 2, 128, 32, 2), (3, 3, 48, 32, 2), (2, 2, 64, 64, 1), (5, 1, 64, 128, 2), (2, 1, 6, 10, 2),
                                             (2, 2, 32, 48, 2), (1, 1, 256, 8, 2)])
@pytest.mark.parametrize("biased", [False, True])
def test_norm_rotation_and_store(biased, H, G, D, DV, planes, dtype):
    """Columns with a bias (or none): queries normed, rotated and multiplied by their head's factor; keys normed, rotated and written with the raw values into
    pages whose values have another size (or none): nothing else of the cache changes."""
    from xpu_serve_b200.ops import lib as ops
    rng = np.random.default_rng(D + DV)
    T, page, eps = 9, 64, 1e-5
    cols = H * D + G * D + (G * DV if planes == 2 else 0)
    x = torch.from_numpy(rng.standard_normal((T, cols + 8))).to(dtype)
    seq_of, positions = [0, 0, 0, 1, 1, 2, 2, 2, 2], [62, 63, 64, 0, 1, 126, 127, 128, 129]
    table = torch.tensor([[3, 1, -1], [5, -1, -1], [0, 2, 4]], dtype=torch.int32)
    pool0 = torch.from_numpy(rng.standard_normal((6, *ops.kv_page_shape(G, page, D, DV, planes)))).to(dtype)
    pool = pool0.clone().cuda()
    w = torch.from_numpy(rng.uniform(0.5, 1.5, D)).float()
    rope = torch.from_numpy(rng.standard_normal((200, D // 2, 2))).float()
    temp = torch.from_numpy(rng.uniform(-1.5, 1.5, H)).float()
    bias = torch.from_numpy(rng.standard_normal(cols + 8)).float() if biased else None
    q = torch.empty(T, H, D, dtype=dtype, device="cuda")
    ops.qk_norm_rope_store(x.cuda()[:, :cols], q, pool, table.cuda(), dev_i32(seq_of), dev_i32(positions), w.cuda(), w.cuda(), rope.cuda(),
                           H, G, D, page, eps, True, v_dim=DV, planes=planes, q_scale=temp.cuda(),
                           bias=bias.cuda() if biased else None)
    xd, r, half = x.double().numpy() + (bias.double().numpy() if biased else 0.0), rope.double().numpy(), D // 2

    def turn(rows):                 # [T, n, D]
        y = plain.unit_rms(rows, eps) * w.double().numpy()
        c, s = r[positions][:, None, :, 0], r[positions][:, None, :, 1]
        return np.concatenate([y[..., :half] * c - y[..., half:] * s, y[..., half:] * c + y[..., :half] * s], -1)

    tol = 1e-5 if dtype == torch.float32 else 1e-2
    want_q = turn(xd[:, :H * D].reshape(T, H, D)) * temp.double().numpy()[:, None]
    assert np.abs(q.double().cpu().numpy() - want_q).max() <= tol * np.abs(want_q).max()
    want_k = turn(xd[:, H * D:(H + G) * D].reshape(T, G, D))
    flat = pool0.clone().view(6, -1)
    k_view, v_view = flat[:, :G * page * D].view(6, G, page, D), flat[:, G * page * D:]
    for t in range(T):
        p = int(table[seq_of[t], positions[t] // page])
        k_view[p, :, positions[t] % page] = torch.from_numpy(want_k[t]).to(dtype)
        if planes == 2:
            v_view.view(6, G, page, DV)[p, :, positions[t] % page] = torch.from_numpy(xd[t, (H + G) * D:cols]).to(dtype).view(G, DV)
    got, want = pool.double().cpu().numpy().reshape(6, -1), flat.double().numpy()
    assert np.abs(got - want).max() <= tol * np.abs(want).max()
    if not biased:
        assert np.array_equal(got[:, G * page * D:], want[:, G * page * D:])      # values as they are
    touched = np.zeros((6, G, page, D), dtype=bool)
    for t in range(T):
        touched[int(table[seq_of[t], positions[t] // page]), :, positions[t] % page] = True
    same = pool0.double().numpy().reshape(6, -1)[:, :G * page * D].reshape(6, G, page, D)
    assert np.array_equal(got[:, :G * page * D].reshape(6, G, page, D)[~touched], same[~touched])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("F", [1, 50, 72, 256, 4096, 8192, 9000])
def test_poly_norm_alone(F, dtype):
    """Rows of ordinary numbers, of tiny ones (where eps decides), of large ones (sixth powers), and a row of zeros."""
    from xpu_serve_b200.ops import lib as ops
    rng = np.random.default_rng(F)
    z = rng.standard_normal((6, F))
    z[1] *= 1e-3
    z[2] *= 300.0
    z[3] = 0.0
    z[4, 0] = 40.0                                        # one entry decides all three sums
    z = torch.from_numpy(z).to(dtype)
    act = torch.tensor([0.7, -0.4, 0.9, 0.21])
    out = torch.empty(6, F, dtype=dtype, device="cuda")
    ops.poly_norm(z.cuda(), act.cuda(), out, 1e-5)
    want = plain.poly_norm(z.double().numpy(), act.double().numpy(), 1e-5)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    gap = np.abs(out.double().cpu().numpy() - want).max(-1) / np.abs(want).max(-1)
    assert (gap <= tol).all(), gap


@pytest.mark.parametrize("E,identity,top,groups,keep", [(5, 1, 2, 2, 1), (14, 4, 5, 3, 2), (7, 2, 3, 3, 2), (8, 0, 1, 1, 1), (40, 24, 6, 8, 3), (60, 4, 8, 4, 4), (200, 56, 16, 16, 2), (60, 4, 29, 2, 1)])
def test_routing_kernel_alone(E, identity, top, groups, keep):
    """Choices and weights against the oracle's wherever the choice is no close call; corrections of both signs, so that open
    groups hold negative choice scores."""
    from xpu_serve_b200.ops import lib as ops
    rng = np.random.default_rng(E)
    T, n = 300, E + identity
    z = torch.from_numpy(rng.standard_normal((T, n + 3)) * 3).float()
    corr = torch.from_numpy(rng.uniform(-0.6, 0.3, n)).float()
    ids = torch.empty(T * top, dtype=torch.int32, device="cuda")
    wts = torch.empty(T * top, dtype=torch.float32, device="cuda")
    ops.moe_route_grouped(z.cuda(), top, ids, wts, experts=n, correction=corr.cuda(), groups=groups, keep=keep, group_top=1, renorm=True,
                          renorm_eps=1e-20, score="softmax", real=E)
    ids, wts = ids.cpu().numpy().reshape(T, top), wts.cpu().numpy().reshape(T, top)
    sure = 0
    for t in range(T):
        want, w, margin = plain.route(z[t, :n].double().numpy(), corr.double().numpy(), top, groups, keep)
        if margin > 1e-5:
            sure += 1
            assert np.array_equal(ids[t], np.where(want >= E, -1, want)), t
            assert np.abs(wts[t] - w).max() < 1e-5
    assert sure > T // 2


def test_weights_of_vanishing_scores():
    """Chosen scores that underflow to nothing give weights of zero, not NaN."""
    from xpu_serve_b200.ops import lib as ops
    z = torch.tensor([[200.0, 0.0, 0.0, 0.0]])
    corr = torch.tensor([-9.0, 0.0, 1.0, 2.0])
    ids = torch.empty(2, dtype=torch.int32, device="cuda")
    wts = torch.empty(2, dtype=torch.float32, device="cuda")
    ops.moe_route_grouped(z.cuda(), 2, ids, wts, correction=corr.cuda(), group_top=1, renorm=True, renorm_eps=1e-20, score="softmax")
    assert ids.tolist() == [3, 2] and wts.tolist() == [0.0, 0.0]


def test_stream_add_alone():
    from xpu_serve_b200.ops import lib as ops
    for T, n in ((5, 44), (3, 45), (1, 7), (300, 64)):
        h, base, row = (torch.randn(*s) for s in ((T, n), (T, n), (n,)))
        for b, r in ((base, row), (None, row), (base, None)):
            d = h.clone().cuda()
            ops.stream_add(d, None if b is None else b.cuda(), None if r is None else r.cuda())
            want = h + (0 if b is None else b) + (0 if r is None else r)
            assert (d.cpu() - want).abs().max() <= 1e-6


def test_the_program_replays_a_trace(folders, tmp_path):
    """bin/trace_run over its standard input, in float32, against the oracle."""
    reqs = requests_for("A", [5, 40, 70])
    steps = tu.tail_trace(reqs, tail=4)
    folder = folders("A", "float32")
    got = tu.collect(steps, tu.run_program(folder, "float32", steps, str(tmp_path / "out"), 512, tiny.CONFIGS["A"]["vocab"]),
                     tiny.CONFIGS["A"]["vocab"])
    ref = reference(folder, reqs)
    gap, where, cos = tu.worst_gap({k: got[k] for k in ref}, ref)
    assert gap <= 1e-5 and cos >= COS["float32"], (gap, where, cos)


# --------------------------------------------------------------------------------------------------------- generation
def plain_greedy(cfg, W, prompt, n):
    seq, out, margins = list(prompt), [], []
    for _ in range(n):
        logits = plain.forward(cfg, W, seq)[-1]
        order = np.argsort(-logits)
        margins.append(min((logits[order[0]] - logits[order[1]]) / np.abs(logits).max(), plain.router_margins(cfg, W, seq).min()))
        out.append(int(order[0]))
        seq.append(out[-1])
    return out, margins


@pytest.mark.parametrize("precision,name", [("f32", "A"), ("f32", "B"), ("bf16", "whole_loop")])
@pytest.mark.parametrize("chunk", [None, 16])
def test_greedy_generation_through_the_engine(folders, chunk, precision, name):
    """The framework's own entry point and scheduler: three unequal prompts as one batch (with `chunk`, prompts in pieces of
    16 tokens), greedy, against the plain implementation run token by token. In float32 every token must be the oracle's; in
    bfloat16 a sequence is followed until the oracle's own choice is a near tie."""
    from xpu_serve_b200 import GenerateRequest, SamplingParams
    from xpu_serve_b200.engine.engine import Engine
    dtype = {"f32": "float32", "bf16": "bfloat16"}[precision]
    folder = folders(name, dtype)
    cfg, W = load_folder(folder)
    kw = {} if chunk is None else {"prefill_chunk": chunk}
    engine = Engine(folder, precision=precision, ctx=256, max_batch=8, **kw)
    prompts = [tiny.prompt(name, n, salt=i) for i, n in enumerate((3, 41, 18))]
    res = engine.generate([GenerateRequest(p, SamplingParams(temperature=0.0), 9, []) for p in prompts])
    followed = 0
    for p, r in zip(prompts, res):
        assert r.finish == "length" and len(r.tokens) == 9
        seq = list(p)
        near = 1e-4 if precision == "f32" else 0.03
        for t in r.tokens:
            logits = plain.forward(cfg, W, seq)[-1]
            order = np.argsort(-logits)
            close = plain.router_margins(cfg, W, seq).min() < CLOSE_CALL[dtype]
            if close or (logits[order[0]] - logits[order[1]]) / np.abs(logits).max() < near:
                break
            assert t == int(order[0]), (len(seq) - len(p), t, int(order[0]))
            followed += 1
            seq.append(t)
    assert followed >= 6, "near ties everywhere; pick other prompts"
    engine.stepper.cache.check()
    assert engine.stepper.cache.slots.held_count == 0


@pytest.mark.parametrize("chunk", [None, 16])
def test_generation_with_experts_in_bfloat16_follows_replay(folders, replayers, chunk):
    """With experts the oracle's choice is a close call too often at 16 bits to follow it for long, so here the engine (prompts
    as captured graphs or in pieces of 16 tokens; decode graphs, one step ahead of the loop) is held against trace replay of
    the same tokens (plain launches): two paths through the same kernels. A token may differ only where replay's own two best
    logits are within a hundredth of the largest."""
    from xpu_serve_b200 import GenerateRequest, SamplingParams
    from xpu_serve_b200.engine.engine import Engine
    folder = folders("B", "bfloat16")
    kw = {} if chunk is None else {"prefill_chunk": chunk}
    engine = Engine(folder, precision="bf16", ctx=256, max_batch=8, **kw)
    prompts = [tiny.prompt("B", n, salt=i) for i, n in enumerate((3, 41, 18))]
    res = engine.generate([GenerateRequest(p, SamplingParams(temperature=0.0), 9, []) for p in prompts])
    rp = replayers("B", "bfloat16")
    same = 0
    for p, r in zip(prompts, res):
        assert r.finish == "length" and len(r.tokens) == 9
        logits = rp.run_step({"step": 0, "entries": [{"id": "g", "tokens": p, "want": [0, len(p) - 1]}], "end": []})[-1]
        for i, t in enumerate(r.tokens):
            order = np.argsort(-logits)
            if t != int(order[0]):
                assert (logits[order[0]] - logits[order[1]]) / np.abs(logits).max() < 1e-2, (i, t, int(order[0]))
                break
            same += 1
            logits = rp.run_step({"step": i + 1, "entries": [{"id": "g", "tokens": [t], "want": [0]}], "end": []})[0]
        rp.run_step({"step": 99, "entries": [], "end": ["g"]})
    assert same >= 16
    engine.stepper.cache.check()
    assert engine.stepper.cache.slots.held_count == 0 and rp.cache.slots.held_count == 0


def test_the_command_line_generates(folders):
    """`bin/xpu-serve run` on a Gararax folder in float32, greedy: the plain implementation's tokens."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    folder = folders("C", "float32")
    cfg, W = load_folder(folder)
    prompt = tiny.prompt("C", 11, salt=91)
    want, margins = plain_greedy(cfg, W, prompt, 8)
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "xpu-serve"), "run", folder, "--prompt", " ".join(map(str, prompt)),
                        "--max-tokens", "8", "--temperature", "0", "--precision", "f32", "--ctx", "128"],
                       capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    res = json.loads(p.stdout.strip().splitlines()[-1])
    assert len(res["tokens"]) == 8
    k = next((i for i, m in enumerate(margins) if m <= 1e-4), 8)
    assert res["tokens"][:k] == want[:k]
