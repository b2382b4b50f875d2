"""The Fosavik decoder against a plain implementation written from the design's equations (``plain_fosavik``):
each mechanism alone, whole models whole, in portions, decoded, mixed, and generation through the engine.

Tiny configurations and random weights are made here; where random weights would hide a fault (a window's edge, the
kept first keys, a far key in either map, the sink, the limit of the feed-forward) rows or weights are scaled so that it
shows.
"""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_fosavik as plain
from plain_qwen3 import read_model_folder
from tiny_configs import random_tokens

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]


def maps(heads, kv_heads, dim, vdim, scale, diff, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def sink(heads, kv_heads, dim, scale, size, keep_first):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "mask": {"size": size, "keep_first": keep_first}}


def recurrence(width, blocks, conv):
    return {"width": width, "blocks": blocks, "conv": conv}


def parallel(left, right, left_scale, right_scale):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def layer(entry, ff=None, limit=None):
    return {**entry, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


# A: sizes in multiples of 8, values twice as wide as a map's keys, a window of two pages that keeps three first keys, a
# reader that follows its source at a distance, a second layer with keys of its own between them.  B: nothing a multiple of
# 8, values narrower and wider than both maps' keys, six query heads on one kv head, more kept keys than the window is
# wide, a convolution of one tap and one of five, three copies of the stream, two readers of one source, a parallel layer
# first and one without feed-forward, sides scaled by negative and large constants.  C: one copy of the stream, one
# attention layer, a window that keeps nothing.
CONFIG_A = {
    "architecture": "Fosavik", "width": 64, "vocab": 200, "max_positions": 400, "streams": 2, "norm": {"eps": 1e-5},
    "layers": [
        layer(maps(4, 2, 16, 32, 0.6, 0.3), 96, 1.5),
        layer(parallel(sink(4, 2, 16, 0.7, 8, 3), recurrence(48, 3, 4), 0.8, 1.3), 72, 0.9),
        layer(maps(2, 2, 8, 24, 0.9, 0.7)),
        layer(mamba(4, 8, 16, 2, 4, 2)),
        layer(maps(4, 2, 16, 32, 0.4, 0.6, kv_from=0), 40, 3.0),
    ],
}
CONFIG_B = {
    "architecture": "Fosavik", "width": 100, "vocab": 131, "max_positions": 370, "streams": 3, "norm": {"eps": 1e-3},
    "layers": [
        layer(parallel(sink(6, 1, 12, 0.9, 5, 7), recurrence(54, 9, 1), -0.7, 1.9)),
        layer(maps(6, 3, 10, 14, 0.5, 0.8), 52, 2.5),
        layer(mamba(5, 12, 6, 5, 3, 3), 33, 0.6),
        layer(maps(6, 3, 10, 14, 0.7, 0.2, kv_from=1), 44, 1.1),
        layer(parallel(sink(3, 3, 10, 1.1, 11, 1), recurrence(40, 1, 5), 1.4, 0.5), 60, 1.0),
        layer(maps(6, 3, 10, 14, 1.0, 0.4, kv_from=1)),
        layer(maps(4, 1, 6, 22, 0.8, 0.5), 28, 4.0),
    ],
}
CONFIG_C = {
    "architecture": "Fosavik", "width": 48, "vocab": 90, "max_positions": 512, "streams": 1, "norm": {"eps": 1e-6},
    "layers": [layer(parallel(sink(2, 1, 24, 0.5, 16, 0), recurrence(32, 2, 2), 1.0, 1.0), 64, 7.0),
               layer(maps(3, 1, 40, 56, 0.3, 0.45), 24, 2.0)],
}
TINY = {"A": (CONFIG_A, 4, 3), "B": (CONFIG_B, 8, 4), "C": (CONFIG_C, 16, 5)}  # name -> (config, page size, seed)


def write_model(folder, raw, seed, std=0.08):
    import kirai_b200  # noqa: F401
    from kirai_b200.registry import config_from_dict
    from kirai_b200.weights import write_random_model

    write_random_model(folder, config_from_dict(raw), seed, std=std, norm_jitter=0.3, dtype=torch.bfloat16)


def tolerance(dtype, reference):
    dtype = {torch.float32: "float32", torch.bfloat16: "bfloat16"}.get(dtype, dtype)
    peak = float(np.abs(np.asarray(reference)).max())
    return 3e-5 * max(1.0, peak) if dtype == "float32" else 0.035 * peak


def close(dtype, got, expected, what):
    got, expected = np.asarray(got, dtype=np.float64), np.asarray(expected, dtype=np.float64)
    assert got.shape == expected.shape, what
    if not got.size:
        return
    worst = float(np.abs(got - expected).max())
    assert worst <= tolerance(dtype, expected), f"{what}: max abs diff {worst} (bound {tolerance(dtype, expected)})"


# --------------------------------------------------------------------------- no GPU
def test_config_reads_every_size_and_round_trips():
    import kirai_b200  # noqa: F401
    from kirai_b200.config.base import ConfigError
    from kirai_b200.registry import config_from_dict, plan_for_config

    for raw in (CONFIG_A, CONFIG_B, CONFIG_C):
        cfg = config_from_dict(raw)
        assert cfg.to_dict() == raw and config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
        plan = plan_for_config(cfg)
        assert plan.max_positions == raw["max_positions"]
        needs, at = plan.cache_needs, 0
        for call, entry in zip(plan.order, raw["layers"]):
            m = entry["mixer"]
            if entry["type"] == "parallel":
                kv, state = needs[at], needs[at + 1]
                left, right = m["left"], m["right"]
                assert (kv.kv_heads, kv.window, kv.keep_first) == (left["kv_heads"], left["mask"]["size"], left["mask"]["keep_first"])
                assert kv.key_dim == kv.value_dim == left["dim"]
                assert state.shape == (right["conv"] * right["width"],) and state.dtype == torch.float32
                at += 2
            elif entry["type"] == "mamba2":
                channels = m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
                assert needs[at].shape == ((m["conv"] - 1) * channels + m["heads"] * m["state"] * m["vdim"],)
                at += 1
            elif "kv_from" in m:
                source = plan.order[m["kv_from"]]
                assert (call.cache, call.write, source.write) == (source.cache, False, True)
            else:
                assert (needs[at].kv_heads, needs[at].key_dim, needs[at].value_dim, needs[at].window) == (m["kv_heads"], 2 * m["dim"], m["vdim"], None)
                at += 1
        assert at == len(needs)
        names = set(plan.weight_specs())
        assert {"embed", "pos", "head", "final.norm", "l0.hc1.in", "l0.hc1.out", "l0.hc1.mix"} <= names
        for i, entry in enumerate(raw["layers"]):
            assert (f"l{i}.mlp.gate" in names) == (f"l{i}.norm2" in names) == (f"l{i}.hc2.mix" in names) == (entry["mlp"] is not None)
            if entry["type"] == "attention":
                assert (f"l{i}.mix.k" in names) == (f"l{i}.mix.v" in names) == ("kv_from" not in entry["mixer"])
            if entry["type"] == "parallel":
                assert f"l{i}.mix.left.v" not in names and {f"l{i}.mix.left.o", f"l{i}.mix.right.o", f"l{i}.mix.left.k.norm"} <= names

    def refused(change):
        bad = json.loads(json.dumps(CONFIG_A))
        change(bad)
        with pytest.raises(ConfigError):
            config_from_dict(bad)

    refused(lambda c: c["layers"][3].update(type="conv"))
    refused(lambda c: c["layers"][0]["mixer"].update(kv_heads=3))
    refused(lambda c: c["layers"][1]["mixer"]["left"].update(vdim=8))
    refused(lambda c: c["layers"][1]["mixer"]["right"].update(blocks=5))
    refused(lambda c: c["layers"][3]["mixer"].update(norm_groups=3))
    refused(lambda c: c["layers"][4]["mixer"].update(kv_from=1))      # no attention layer
    refused(lambda c: c["layers"][4]["mixer"].update(kv_from=4))      # not an earlier one
    refused(lambda c: c["layers"][4]["mixer"].update(kv_from=2))      # other head sizes
    refused(lambda c: c["layers"][0]["mixer"].update(kv_from=4))
    refused(lambda c: c["layers"][0]["mlp"].update(limit=0.0))
    refused(lambda c: c["layers"][0]["mlp"].update(kind="moe"))
    refused(lambda c: c.pop("streams"))


def test_plain_forms_worked_by_hand():
    """The plain functions on numbers small enough to check by eye."""
    w = {"c.in": torch.tensor([1.0, -2.0]), "c.out": torch.tensor([0.5, 3.0]), "c.mix": torch.tensor([[1.0, 10.0], [100.0, 1000.0]])}
    xs = torch.tensor([[[1.0]], [[2.0]]])  # two copies, one token, width one
    assert float(plain.streams_read(xs, w, "c.")) == 1.0 - 4.0
    # to copy 0: 1 * 1 + 100 * 2 + 0.5 y; to copy 1: 10 * 1 + 1000 * 2 + 3 y
    assert plain.streams_update(xs, torch.tensor([[2.0]]), w, "c.").flatten().tolist() == [202.0, 2016.0]
    p = plain.softmax_with_sink(torch.tensor([[0.0, 0.0, float("-inf")], [3.0, float("-inf"), float("-inf")]], dtype=torch.float64))
    assert torch.allclose(p[0], torch.tensor([1 / 3, 1 / 3, 0.0], dtype=torch.float64))
    assert abs(float(p[1, 0]) - np.exp(3.0) / (1.0 + np.exp(3.0))) < 1e-12
    assert plain.visible_keys(12, 4, 2)[11].tolist() == [True, True] + [False] * 6 + [True] * 4
    taps = torch.tensor([[1.0, 10.0, 100.0]])
    assert plain.causal_convolution(torch.tensor([[1.0], [2.0], [3.0]]), taps, torch.tensor([0.5])).flatten().tolist() == [100.5, 210.5, 321.5]
    # two blocks of two channels, each through its own [out, in] matrix
    weight = torch.tensor([[[1.0, 2.0], [3.0, 4.0]], [[0.0, 1.0], [1.0, 0.0]]])
    assert plain.block_product(torch.tensor([[1.0, 1.0, 5.0, 7.0]]), weight, torch.zeros(2, 2)).flatten().tolist() == [3.0, 7.0, 7.0, 5.0]


# ------------------------------------------------------------------------ parts alone
def _mixer(entry, width, eps=1e-5):
    """The framework's mixer of one configured layer (its tensors under ``a.``) and the layer as config.json holds it."""
    import kirai_b200  # noqa: F401
    from kirai_b200.config.fosavik import FosavikConfig
    from kirai_b200.models.fosavik import mixer_for_layer

    raw = {"architecture": "Fosavik", "width": width, "vocab": 8, "max_positions": 8, "streams": 2, "norm": {"eps": eps},
           "layers": [layer(entry)]}
    cfg = FosavikConfig.from_dict(raw)
    return mixer_for_layer(cfg, cfg.layers[0], "a."), raw["layers"][0]["mixer"]


def _needs(part):
    need = part.cache_need()
    return list(need) if isinstance(need, tuple) else [need]


def _view(part, session):
    if isinstance(part.cache_need(), tuple):
        return tuple(session.cache.layer_view(i) for i in range(len(part.cache_need())))
    return session.cache.layer_view(0)


def _run_together(part, session, xs, steps, forward=None):
    """The part's output rows for several requests (``xs``: name -> rows [T, width]) under a schedule: ``steps`` is a
    list of steps, each a list of (name, count) that run as one batch.  A request is closed after its last row."""
    forward = forward or (lambda x, batch: part.forward(x, batch, _view(part, session)))
    names = list(xs)
    offset, table = {}, []
    for name in names:
        offset[name] = sum(t.shape[0] for t in table)
        table.append(xs[name])
    table = torch.cat(table)
    done = {name: 0 for name in names}
    out = None
    for step in steps:
        runs = [(name, list(range(offset[name] + done[name], offset[name] + done[name] + count))) for name, count in step]
        batch = session.batch(runs)
        rows = batch.token_ids.cpu().long()
        y = forward(table[rows].cuda(), batch).float().cpu()
        if out is None:
            out = torch.zeros((table.shape[0], y.shape[1]))
        out[rows] = y
        session.commit()
        for name, count in step:
            done[name] += count
            if done[name] == xs[name].shape[0]:
                session.cache.close(session.requests.pop(name))
    assert all(done[name] == xs[name].shape[0] for name in names)
    return {name: out[offset[name] : offset[name] + xs[name].shape[0]] for name in names}


def _run_part(part, session, x, cuts, forward=None):
    return _run_together(part, session, {"s": x}, [[("s", size)] for size in cuts], forward)["s"]


def CUTS(n):
    return [n], [37, 2, 19, 1, 1, 3, n - 63], [n - 10] + [1] * 10, [2] * (n // 2) + [1] * (n % 2), [1] * n


UNEQUAL = [[("p", 40), ("q", 2)], [("p", 1), ("q", 20)], [("p", 1), ("q", 1)], [("q", 10), ("p", 28)],      # p and q end here
           [("r", 7), ("s", 1)], [("r", 1), ("s", 30)], [("s", 1), ("r", 1)], [("s", 16)],                   # r ends, then s
           [("t", 1)], [("t", 1)]]


def _unequal_rows(width, seed, dtype):
    g = torch.Generator().manual_seed(seed)
    return {name: (torch.randn((n, width), generator=g) * 1.5).to(dtype) for name, n in (("p", 70), ("q", 33), ("r", 9), ("s", 48), ("t", 2))}


# ---- copies of the stream ---------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("copies,width", [(1, 64), (2, 100), (3, 7), (4, 2048 + 24), (4, 4096), (3, 8192), (5, 96), (8, 33), (4, 8200)])
def test_streams_updated_read_and_normed(dtype, copies, width):
    """Two sub-layers in a row on copies that are still equal at first, then the chosen rows of the copies' sum; a norm that
    does not take streams gives what its own kernel makes of the reading."""
    from part_helpers import load_part
    from kirai_b200.parts import LayerNorm, RMSNorm, StreamConnection
    from kirai_b200.parts.base import StreamUpdate

    T, eps = 11, 1e-4
    one, two = StreamConnection("a.", copies), StreamConnection("b.", copies)
    norm, other = RMSNorm("n", width, eps), LayerNorm("m", width, eps)
    w = {}
    for seed, part in enumerate((one, two, norm, other)):
        w.update(load_part(part, dtype, seed=seed + width))
    w = {k: v.double() for k, v in w.items()}
    g = torch.Generator().manual_seed(copies)
    x, y1, y2 = (torch.randn((T, width), generator=g) * s for s in (1.0, 3.0, 0.5))
    xs = torch.stack([x.double()] * copies)

    def normed(u, name="n"):
        return plain.rms_norm(u, w[name], eps)

    resid = x.cuda()
    rows, resid = one.enter(resid, None, norm)
    assert resid.dim() == 2 and rows.dtype == dtype
    close(dtype, rows.float().cpu(), normed(plain.streams_read(xs, w, "a.")), "first reading")
    left = one.leave(y1.cuda())
    assert isinstance(left, StreamUpdate)
    before = resid.clone()
    rows, resid = two.enter(resid, left, norm)
    assert resid.shape == (T, copies, width) and torch.equal(before, x.cuda())
    xs = plain.streams_update(xs, y1.double(), w, "a.")
    close(torch.float32, resid.cpu().permute(1, 0, 2), xs, "copies after the first update")
    close(dtype, rows.float().cpu(), normed(plain.streams_read(xs, w, "b.")), "second reading")
    left = two.leave(y2.cuda())
    kept = resid.clone()
    wanted = torch.tensor([9, 0, 4], dtype=torch.int32)
    after = plain.streams_update(xs, y2.double(), w, "b.")
    picked = norm.add_forward_rows(resid, left, wanted.cuda())
    assert torch.equal(kept, resid)  # chosen rows leave the copies alone
    close(dtype, picked.float().cpu(), normed(after.sum(0))[wanted.long()], "rows of the sum")
    rows, same = one.enter(resid, left, norm)
    assert same.data_ptr() == resid.data_ptr()  # in place
    close(torch.float32, same.cpu().permute(1, 0, 2), after, "copies after the second update")
    # another norm, after one more update
    rows, same = one.enter(same, two.leave(y1.cuda()), other)
    after = plain.streams_update(after, y1.double(), w, "b.")
    u = plain.streams_read(after, w, "a.")
    centred = u - u.mean(-1, keepdim=True)
    close(dtype, rows.float().cpu(), centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * w["m"], "layer norm of the reading")


@pytest.mark.gpu
def test_a_last_norm_of_another_kind_reads_the_copies_sum():
    from part_helpers import DEV, load_part, runtime
    from kirai_b200.models.plan import DecoderModel, LayerCall, ModelPlan
    from kirai_b200.parts import Block, Embedding, GatedMLP, LayerNorm, OutputHead, RMSNorm, StreamConnection  # noqa: F401
    from kirai_b200.parts.base import StreamUpdate

    norm, head = LayerNorm("n", 24, 1e-5), OutputHead("h", 16, 24)
    block = Block(RMSNorm("n1", 24, 1e-5), _mixer(maps(2, 1, 4, 8, 1.0, 0.5), 24)[0], None, None, arrangement="streams",
                  connection1=StreamConnection("c.", 3))
    plan = ModelPlan(Embedding("e", 16, 24), [block], [LayerCall(block=0, cache=0)], norm, head, 16, 24)
    model = DecoderModel(plan, runtime(torch.float32))
    w = {}
    for part in (norm, head):
        w.update(load_part(part, torch.float32, seed=4))
    g = torch.Generator().manual_seed(0)
    streams, y = torch.randn((5, 3, 24), generator=g), torch.randn((5, 24), generator=g)
    mix, add = torch.randn((3, 3), generator=g), torch.randn(3, generator=g)
    got = model.logits(streams.to(DEV), StreamUpdate(y.to(DEV), mix.to(DEV), add.to(DEV)), torch.tensor([4, 1], dtype=torch.int32, device=DEV))
    total = (torch.einsum("tfw,fg->tw", streams.double(), mix.double()) + add.double().sum() * y.double())[[4, 1]]
    centred = total - total.mean(-1, keepdim=True)
    expected = (centred / torch.sqrt((centred ** 2).mean(-1, keepdim=True) + 1e-5) * w["n"].double()) @ w["h"].double().T
    close(torch.float32, got.cpu(), expected, "logits")


def test_blocks_refuse_connections_that_do_not_fit():
    from kirai_b200.parts import Block, RMSNorm, StreamConnection, SwiGLU

    norm, ffn = RMSNorm("n", 8, 1e-5), SwiGLU("m.", 8, 8)
    mixer, c = _mixer(maps(1, 1, 4, 4, 1.0, 0.5), 8)[0], StreamConnection("c.", 2)
    Block(norm, mixer, None, None, arrangement="streams", connection1=c)
    for kwargs in (dict(arrangement="streams"), dict(arrangement="pre_norm", connection1=c),
                   dict(arrangement="streams", connection1=c, connection2=c)):
        with pytest.raises(ValueError):
            Block(norm, mixer, None, None, **kwargs)
    with pytest.raises(ValueError):
        Block(norm, mixer, norm, ffn, arrangement="streams", connection1=c)


# ---- attention as the difference of two maps ----------------------------------------------------------------------------
MAPS_CASES = [  # (heads, kv heads, dim, vdim, scale, diff), width, page size
    ((4, 2, 16, 32, 0.6, 0.3), 64, 4), ((6, 3, 10, 14, 0.5, 0.8), 100, 8), ((4, 1, 6, 22, 0.8, 0.5), 60, 16), ((2, 2, 64, 128, 0.125, 0.9), 96, 16),
    ((8, 1, 32, 64, 0.2, 0.1), 64, 64), ((3, 1, 64, 48, 0.15, 0.6), 40, 16), ((2, 1, 128, 256, 0.08, 0.4), 48, 16),
    ((2, 1, 136, 40, 0.08, 0.4), 32, 4), ((12, 1, 24, 40, 0.2, 0.7), 48, 2),
]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case,width,page", MAPS_CASES, ids=lambda c: "x".join(map(str, c[:4])) if isinstance(c, tuple) else str(c))
def test_two_maps_whole_in_portions_and_one_by_one(dtype, case, width, page):
    from part_helpers import Session, load_part
    from kirai_b200.weights.random_init import random_tensors

    part, raw = _mixer(maps(*case), width)
    tensors = random_tensors(part.weight_specs(), sum(case[:4]), std=0.12, dtype=torch.bfloat16)
    for name in ("a.lq1", "a.lk1", "a.lq2", "a.lk2"):
        tensors[name] = (tensors[name].float() * (4.0 if name.endswith("1") else 2.0)).to(torch.bfloat16)  # a lambda that is not ``diff``
    w = {k: v.double() for k, v in load_part(part, dtype, tensors=tensors).items()}
    assert abs(float(plain.map_weight(w, raw, "a.")) - part.factor) < 1e-9
    tokens = 150
    x = (torch.randn((tokens, width), generator=torch.Generator().manual_seed(width)) * 1.5).to(dtype)
    expected = plain.two_map_attention(x.double(), w, raw, "a.", 1e-5, plain.keys_and_values(x.double(), w, raw, "a."))
    session = Session([part.cache_need()], dtype, page_size=page, num_pages=-(-tokens // page) + 1, num_slots=2)
    for cuts in CUTS(tokens):
        close(dtype, _run_part(part, session, x, cuts), expected, f"cut as {cuts[:4]}...")
        assert all(pool.free_pages == session.cache.num_pages for pool in session.cache.tables.pools)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_stands_out_in_each_map(dtype):
    """Queries that are opposed to the keys in one map only, and late tokens that are minus three times an early one: the
    early token takes that map's whole weight, hundreds of keys away, across page borders, in a prompt and decoded.
    Taking the other map's keys, or the maps in the other order, is far outside the bound."""
    from part_helpers import Session, load_part
    from kirai_b200.weights.random_init import random_tensors

    heads, kv_heads, dim, vdim, width, page, total = 4, 2, 32, 24, 56, 8, 420
    for one in (0, 1):
        part, raw = _mixer(maps(heads, kv_heads, dim, vdim, 0.12, 0.55), width)
        tensors = random_tensors(part.weight_specs(), 9 + one, std=0.1, dtype=torch.bfloat16)
        k = tensors["a.k"].view(kv_heads, 2, dim, width)
        q = tensors["a.q"].view(heads, 2, dim, width).clone()
        q[:, one] = (-k[:, one]).repeat_interleave(heads // kv_heads, dim=0)
        tensors["a.q"] = q.reshape(heads * 2 * dim, width)
        w = {name: v.double() for name, v in load_part(part, dtype, tensors=tensors).items()}
        x = torch.randn((total, width), generator=torch.Generator().manual_seed(one)).to(dtype)
        pairs = [(0, 100), (7, 200), (8, 255), (15, 256), (1, 330), (64, 390), (63, 401), (0, 419)]  # the last four are decoded
        for early, late in pairs:
            x[late] = -3.0 * x[early]
        kv = plain.keys_and_values(x.double(), w, raw, "a.")
        expected = plain.two_map_attention(x.double(), w, raw, "a.", 1e-5, kv)
        rows = [late for _, late in pairs]
        swapped = plain.two_map_attention(x.double(), w, raw, "a.", 1e-5, (kv[0].flip(2), kv[1]))
        assert float((swapped - expected)[rows].abs().max()) > 3 * tolerance(dtype, expected.numpy())
        session = Session([part.cache_need()], dtype, page_size=page, num_pages=-(-total // page) + 1, num_slots=2)
        for cuts in ([total], [300] + [1] * 120, [99, 2, 150, 69] + [1] * 50 + [2] * 25):
            close(dtype, _run_part(part, session, x, cuts), expected, f"map {one}, cut as {cuts[:4]}...")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case,width,page", [((4, 2, 16, 32), 64, 4), ((6, 3, 10, 14), 100, 8), ((3, 1, 24, 80), 40, 16)], ids=["a", "b", "c"])
def test_a_layer_that_reads_an_earlier_layers_keys_and_values(dtype, case, width, page):
    """The source's call and the reader's call in the same step, the reader with rows, queries, scale, diff and lambda of
    its own; in batches of unequal requests on reused pages."""
    from part_helpers import Session, load_part
    from kirai_b200.parts import TwoMapAttention

    heads, kv_heads, dim, vdim = case
    source, raw = _mixer(maps(heads, kv_heads, dim, vdim, 0.5, 0.3), width)
    reader = TwoMapAttention("b.", width, heads, kv_heads, dim, vdim, 0.8, 0.6, 1e-5, reads_only=True, out_dtype=torch.float32)
    w = {k: v.double() for k, v in {**load_part(source, dtype, seed=1), **load_part(reader, dtype, seed=2)}.items()}
    assert not {"b.k", "b.v"} & set(w)
    xs = _unequal_rows(width, page, dtype)
    shift = torch.randn(width, generator=torch.Generator().manual_seed(5))
    expected = {}
    for name, x in xs.items():
        x = x.double()
        y = (x + shift.double()).to(dtype).double()
        kv = plain.keys_and_values(x, w, raw, "a.")
        expected[name] = plain.two_map_attention(y, w, {**raw, "scale": 0.8, "diff": 0.6}, "b.", 1e-5, kv)
    session = Session([source.cache_need()], dtype, page_size=page, num_pages=-(-70 // page) - (-48 // page), num_slots=2)
    assert source.cache_need() == reader.cache_need()

    def forward(x, batch):
        view = session.cache.layer_view(0)
        source.forward(x, batch, view, True)
        return reader.forward((x.double() + shift.double().cuda()).to(dtype), batch, view, False)

    got = _run_together(reader, session, xs, UNEQUAL, forward)
    for name in xs:
        close(dtype, got[name], expected[name], f"request {name}")
    with pytest.raises(ValueError):
        reader.forward(xs["t"].cuda(), None, None, True)


# ---- attention with a sink, kept first keys, and values that are the keys ----------------------------------------------------
SINK_CASES = [  # (heads, kv heads, dim, scale, window, kept first keys), width, page size
    ((4, 2, 16, 0.7, 8, 3), 64, 4), ((6, 1, 12, 0.9, 5, 7), 100, 8), ((2, 2, 32, 0.4, 16, 0), 40, 16), ((3, 3, 10, 1.1, 11, 1), 30, 2),
    ((4, 2, 72, 0.125, 33, 4), 64, 16), ((8, 2, 128, 0.09, 41, 17), 96, 16), ((2, 1, 24, 0.3, 1, 2), 48, 8), ((2, 1, 200, 0.1, 64, 5), 32, 64),
]


def _left_side(case, width, eps=1e-5):
    """The attention side with its own outer products (``alone``: not sharing them with a second side)."""
    from kirai_b200.parts import GQAttention

    heads, kv_heads, dim, scale, size, keep = case
    return GQAttention("a.left.", width, heads, kv_heads, dim, None, window=size, scale=scale, qk_norm_eps=eps,
                       names={"q": "q", "k": "k", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"}, head_gate="g", keep_first=keep,
                       keys_as_values=True, sink=0.0, out_dtype=torch.float32), sink(*case)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case,width,page", SINK_CASES, ids=lambda c: "x".join(map(str, c)) if isinstance(c, tuple) else str(c))
def test_sink_attention_whole_in_portions_and_one_by_one(dtype, case, width, page):
    """150 tokens under every cut, on a pool with no page to spare, so that pages the window gave back are used again; the
    pages of the kept first keys stay.  Leaving the sink out, or norming the values, is far outside the bound."""
    from part_helpers import Session, load_part

    part, raw = _left_side(case, width)
    w = {k: v.double() for k, v in load_part(part, dtype, seed=13).items()}
    assert "a.left.v" not in w
    tokens = 150
    x = (torch.randn((tokens, width), generator=torch.Generator().manual_seed(width)) * 1.5).to(dtype)
    expected = plain.sink_attention(x.double(), w, raw, "a.left.", 1e-5)
    with_sink = plain.softmax_with_sink
    try:
        plain.softmax_with_sink = lambda scores: torch.softmax(scores, dim=-1)
        without = plain.sink_attention(x.double(), w, raw, "a.left.", 1e-5)
    finally:
        plain.softmax_with_sink = with_sink
    assert float((without - expected).abs().max()) > 1.5 * tolerance(dtype, expected.numpy())
    session = Session([part.cache_need()], dtype, page_size=page, num_pages=-(-tokens // page) + 1, num_slots=2)
    for cuts in CUTS(tokens):
        close(dtype, _run_part(part, session, x, cuts), expected, f"cut as {cuts[:4]}...")
        assert all(pool.free_pages == session.cache.num_pages for pool in session.cache.tables.pools)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep,page", [(16, 3, 4), (21, 6, 8), (64, 1, 16), (7, 9, 4)])
def test_keys_at_the_windows_edge_and_the_kept_first_keys_stand_out(dtype, size, keep, page):
    """Queries opposed to the keys, large norm weights, and pairs of (early, late) tokens of which late puts its weight on
    early if it sees it: early just inside the window, just outside, the last kept key and the first that is not kept, in
    a prompt and decoded.  A window or a count of kept keys that is off by one is far outside the bound."""
    from part_helpers import Session, load_part
    from kirai_b200.weights.random_init import random_tensors

    case, width = (4, 2, 64, 0.6, size, keep), 48
    part, raw = _left_side(case, width)
    tensors = random_tensors(part.weight_specs(), 21, std=0.08, norm_jitter=0.1, dtype=torch.bfloat16)
    k = tensors["a.left.k"].view(2, 64, -1)
    tensors["a.left.q"] = (-k).repeat_interleave(2, dim=0).reshape(4 * 64, -1)
    tensors["a.left.q.norm"] = torch.full((64,), 0.5, dtype=torch.bfloat16)
    tensors["a.left.k.norm"] = torch.full((64,), 0.5, dtype=torch.bfloat16)
    w = {name: v.double() for name, v in load_part(part, dtype, tensors=tensors).items()}
    total = 300
    x = torch.randn((total, width), generator=torch.Generator().manual_seed(size)).to(dtype)
    pairs = [(100 - (size - 1), 100), (130 - size, 130), (keep - 1, 150), (keep, 170),                 # in a prompt
             (250 - (size - 1), 250), (270 - size, 270), (keep - 1, 285), (keep, 295), (0, 299)]      # decoded
    for early, late in pairs:
        x[late] = -3.0 * x[early]
    expected = plain.sink_attention(x.double(), w, raw, "a.left.", 1e-5)
    bound = tolerance(dtype, expected.numpy())
    late_rows = [late for _, late in pairs]
    for other_size, other_keep in ((size + 1, keep), (size - 1, keep), (size, keep + 1), (size, keep - 1)):
        if other_size < 1 or other_keep < 0:
            continue
        other = plain.sink_attention(x.double(), w, {**raw, "mask": {"size": other_size, "keep_first": other_keep}}, "a.left.", 1e-5)
        assert float((other - expected)[late_rows].abs().max()) > 3 * bound, (other_size, other_keep)
    session = Session([part.cache_need()], dtype, page_size=page, num_pages=-(-total // page) + 1, num_slots=2)
    for cuts in ([total], [200] + [1] * 100, [99, 2, 30, 69] + [1] * 50 + [2] * 25):
        close(dtype, _run_part(part, session, x, cuts), expected, f"cut as {cuts[:4]}...")


@pytest.mark.gpu
@pytest.mark.parametrize("group,dim", [(2, 64), (1, 128), (12, 72), (3, 40), (4, 200)])
def test_a_sink_per_head_in_every_attention_kernel(group, dim):
    """Sinks far below, at and far above the scores, one per head, through the two prompt kernels, the plain kernel and the
    decode kernels with one range, ranges merged in a cluster, ranges merged by a second kernel, and the balanced form."""
    from kirai_b200.csrc import ops

    g = torch.Generator().manual_seed(group * dim)
    kv_heads, page, lens = 2, 16, [300, 17, 1, 129]
    heads = kv_heads * group
    pages = [-(-n // page) for n in lens]
    table = torch.zeros((len(lens), max(pages)), dtype=torch.int32)
    order, at = torch.randperm(sum(pages), generator=g).int(), 0
    for r, n in enumerate(pages):
        table[r, :n] = order[at : at + n]
        at += n
    cache = torch.randn((sum(pages), 2, kv_heads, page, dim), generator=g).to(torch.bfloat16)
    q = (torch.randn((len(lens), heads, dim), generator=g) * 1.5).to(torch.bfloat16)
    sinks = torch.linspace(-60.0, 12.0, heads)
    sinks[0] = 0.0
    scale = dim ** -0.5
    for window, keep in ((None, 0), (20, 3)):
        expected = torch.zeros((len(lens), heads, dim), dtype=torch.float64)
        for r, n in enumerate(lens):
            rows = cache[table[r, : pages[r]].long()].double()
            k, v = (rows[:, i].permute(1, 0, 2, 3).reshape(kv_heads, -1, dim)[:, :n] for i in (0, 1))
            see = torch.ones(n, dtype=torch.bool) if window is None else plain.visible_keys(n, window, keep)[n - 1]
            for h in range(heads):
                s = (k[h // group] @ q[r, h].double() * scale)[see]
                weights = torch.softmax(torch.cat([s, sinks[h : h + 1].double()]), dim=0)[:-1]
                expected[r, h] = weights @ v[h // group][see]
        dev = dict(cache=cache.cuda(), block_table=table.cuda())
        context = torch.tensor(lens, dtype=torch.int32).cuda()
        common = dict(window=window, scale=scale, keep_first=keep, sinks=sinks.cuda())
        starts = torch.arange(len(lens) + 1, dtype=torch.int32).cuda()
        results = {"plain": ops.paged_attention_plain(q.cuda(), dev["cache"], dev["block_table"], starts[:-1].contiguous(), context - 1,
                                                      **common),
                   "prompt, mma": ops.attention_prefill(q.cuda(), dev["cache"], dev["block_table"], starts, context, 1, tcgen05=False, **common)}
        if ops.attention_prefill_takes_tcgen05(heads, kv_heads, dim, page):
            results["prompt, tcgen05"] = ops.attention_prefill(q.cuda(), dev["cache"], dev["block_table"], starts, context, 1, tcgen05=True,
                                                               **common)
        for splits in (1, 2, 3, 7):
            results[f"decode, {splits} ranges"] = ops.attention_decode(q.cuda(), dev["cache"], dev["block_table"], context, num_splits=splits,
                                                                       **common)
        for ctas in (3, 40):
            results[f"decode, balanced on {ctas}"] = ops.attention_decode_balanced(q.cuda(), dev["cache"], dev["block_table"], context,
                                                                                   ctas=ctas, **common)
        # the 32-bit kernel on the same numbers
        exact = ops.paged_attention_plain(q.float().cuda(), cache.float().cuda(), dev["block_table"], starts[:-1].contiguous(), context - 1,
                                          **common)
        close(torch.float32, exact.cpu().view(expected.shape), expected, f"32-bit, window {window}")
        for name, got in results.items():
            diff = float((got.float().cpu().view(expected.shape).double() - expected).abs().max())
            assert diff <= 0.02 * float(expected.abs().max()), (name, window, diff)
    ops.check_device_errors(torch.device("cuda", 0))


# ---- the gated linear recurrence ------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("channels,block", [(48, 16), (33, 11), (300, 60)])
def test_convolution_rows_kept_rows_and_pairs(taps, channels, block):
    """Unequal requests in one step from kept rows that are not zero: the rows, the rows as two bfloat16 numbers, and the
    kept rows after the step, with and without the bias on what enters and the silu."""
    from part_helpers import Session
    from kirai_b200.parts.base import StateNeed
    from kirai_b200.csrc import ops

    gen = torch.Generator().manual_seed(taps * channels)
    lens, offset = [9, 2, 1, 20, 3], 5
    L = offset + max(1, (taps - 1) * channels)
    session = Session([StateNeed((L,), torch.float32)], torch.float32, page_size=4, num_pages=4, num_slots=8)
    batch = session.batch([(f"r{i}", n) for i, n in enumerate(lens)])
    T = sum(lens)
    wide = torch.randn((T, channels + 3), generator=gen)
    x = wide[:, 3:]
    weight, bias, in_bias = torch.randn((channels, taps), generator=gen), torch.randn(channels, generator=gen), torch.randn(channels, generator=gen)
    state0 = torch.randn((8, L), generator=gen)
    starts = batch.query_start.cpu().tolist()
    for silu, entering in ((False, in_bias), (True, None)):
        st = state0.clone().cuda()
        out, pair = ops.conv_rows(wide.cuda()[:, 3:], weight.cuda(), bias.cuda(), st, offset, batch, silu=silu,
                                  in_bias=None if entering is None else entering.cuda(), pair_block=block, pair_tokens=128)
        assert torch.equal(st.cpu()[:, :offset], state0[:, :offset])
        parts = pair.cpu()[:, :T].float()
        rebuilt = (parts[..., :block].double() + parts[..., block:].double()).permute(1, 0, 2).reshape(T, channels)
        assert float((rebuilt - out.cpu().double()).abs().max()) <= 2.0 ** -15 * float(out.abs().max())
        for r, (first, n) in enumerate(zip(starts, np.diff(starts))):
            slot = int(batch.slots[r])
            kept = state0[slot, offset : offset + (taps - 1) * channels].view(taps - 1, channels).double()
            rows = x[first : first + n].double() + (0.0 if entering is None else entering.double())
            padded = torch.cat([kept, rows])
            expected = bias.double() + sum(padded[j : j + n] * weight[:, j].double() for j in range(taps))
            close(torch.float32, out.cpu()[first : first + n], plain.silu(expected) if silu else expected, f"rows of request {r}")
            after = st.cpu()[slot, offset : offset + (taps - 1) * channels].view(taps - 1, channels)
            close(torch.float32, after, padded[n:], f"kept rows of request {r}")


@pytest.mark.gpu
@pytest.mark.parametrize("blocks,block,tokens", [(3, 64, 300), (2, 100, 257), (5, 12, 40), (1, 256, 513), (4, 8, 256)])
def test_block_products_do_not_round_their_input(blocks, block, tokens):
    """The gates' products from rows split in two bfloat16 numbers and in 32-bit multiply-adds: both far closer to the
    exact product than one rounding of the rows to bfloat16 would leave them."""
    from kirai_b200.csrc import ops

    gen = torch.Generator().manual_seed(block)
    u = torch.randn((tokens, blocks * block), generator=gen) * 2.0
    weight = torch.randn((blocks, 2 * block, block), generator=gen).to(torch.bfloat16)
    exact = torch.einsum("tbi,boi->tbo", u.double().view(tokens, blocks, block), weight.double())
    rounded = torch.einsum("tbi,boi->tbo", u.to(torch.bfloat16).double().view(tokens, blocks, block), weight.double())
    plain_error = float((rounded - exact).abs().max())
    got = ops.block_product(u.cuda(), weight.float().cuda(), blocks).cpu().view(tokens, blocks, 2 * block)
    assert float((got.double() - exact).abs().max()) < plain_error / 100.0
    padded = -(-tokens // 128) * 128
    high = u.to(torch.bfloat16)
    low = (u - high.float()).to(torch.bfloat16)
    pair = torch.zeros((blocks, padded, 2 * block), dtype=torch.bfloat16)
    pair[:, :tokens, :block] = high.view(tokens, blocks, block).permute(1, 0, 2)
    pair[:, :tokens, block:] = low.view(tokens, blocks, block).permute(1, 0, 2)
    stacked = torch.cat([weight, weight], dim=2).reshape(blocks * 2 * block, 2 * block).contiguous().cuda()
    for matrix in [stacked] + ([ops.tile_weight(stacked)] if (2 * block) % 128 == 0 else []):
        got = ops.block_product_pairs(pair.cuda(), matrix).cpu()[:, :tokens].permute(1, 0, 2)
        assert float((got.double() - exact).abs().max()) < plain_error / 50.0


@pytest.mark.gpu
@pytest.mark.parametrize("out_dtype", DTYPES)
@pytest.mark.parametrize("blocks,block", [(3, 11), (2, 64), (1, 5000)])
def test_scan_of_unequal_requests_from_states_that_are_not_zero(out_dtype, blocks, block):
    """Runs of 1, 7, 8, 9, 33, 256, 257 and 1,300 tokens in one step, gates that hold and that forget, both layouts of the
    gates' rows, an output that is a run of columns of a wider buffer."""
    from part_helpers import Session
    from kirai_b200.parts.base import StateNeed
    from kirai_b200.csrc import ops

    gen = torch.Generator().manual_seed(block)
    lens, W, offset = ([1, 7, 8, 9, 33, 256, 257, 1300] if block < 1000 else [1, 9, 300]), blocks * block, 6
    session = Session([StateNeed((offset + W,), torch.float32)], torch.float32, page_size=4, num_pages=4, num_slots=8)
    batch = session.batch([(f"r{i}", n) for i, n in enumerate(lens)])
    T = sum(lens)
    u, branch = torch.randn((T, W), generator=gen), torch.randn((T, W + 2), generator=gen)
    gates = torch.randn((T, blocks, 2 * block), generator=gen) * 2.0
    rb, ib, bb = (torch.randn(W, generator=gen) for _ in range(3))
    rate = -8.0 * torch.linspace(1e-5, 3.0, W)  # from almost nothing forgotten in a thousand tokens to everything at once
    state0 = torch.randn((8, offset + W), generator=gen) * 3.0
    results = []
    for rows in (gates.reshape(T, -1), torch.cat([gates.permute(1, 0, 2), torch.full((blocks, 20, 2 * block), float("nan"))], dim=1).contiguous()):
        st = state0.clone().cuda()
        buffer = torch.zeros((T, W + 16), dtype=out_dtype).cuda()
        ops.real_gated_scan(u.cuda(), rows.cuda(), block, branch.cuda()[:, 2:], rb.cuda(), ib.cuda(), bb.cuda(), rate.cuda(), st, offset, batch,
                            buffer[:, 16:], 0.7)
        assert float(buffer[:, :16].abs().max()) == 0.0 and torch.equal(st.cpu()[:, :offset], state0[:, :offset])
        results.append((buffer[:, 16:].float().cpu(), st.cpu()))
    starts = batch.query_start.cpu().tolist()
    r = torch.sigmoid(gates[..., :block].double().reshape(T, W) + rb.double())
    i = torch.sigmoid(gates[..., block:].double().reshape(T, W) + ib.double())
    log_a = rate.double() * r
    a, b = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u.double()
    gate = plain.gelu_tanh(branch[:, 2:].double() + bb.double())
    for k, (first, n) in enumerate(zip(starts, np.diff(starts))):
        S = state0[int(batch.slots[k]), offset:].double()
        rows = []
        for t in range(first, first + n):
            S = a[t] * S + b[t]
            rows.append(0.7 * S * gate[t])
        for name, (out, st) in zip(("token by token", "block by block"), results):
            got, want = out[first : first + n].double(), torch.stack(rows)
            bound = 5e-5 if out_dtype == torch.float32 else 0.006
            assert float((got - want).abs().max()) <= bound * float(want.abs().max()), (name, k)
            assert float((st[int(batch.slots[k]), offset:].double() - S).abs().max()) <= 5e-5 * max(1.0, float(S.abs().max())), (name, k)


RECURRENCE_CASES = [(48, 3, 4, 64), (54, 9, 1, 100), (40, 1, 5, 30), (256, 2, 4, 96), (128, 8, 2, 40), (36, 2, 3, 24)]  # width, blocks, taps, hidden


def _recurrence_part(case):
    from kirai_b200.parts import GatedLinearRecurrence

    width, blocks, taps, hidden = case
    return GatedLinearRecurrence("a.right.", hidden, width, blocks, taps, out_dtype=torch.float32), recurrence(width, blocks, taps)


def _recurrence_tensors(part, seed):
    from kirai_b200.weights.random_init import random_tensors

    tensors = random_tensors(part.weight_specs(), seed, std=0.15, dtype=torch.bfloat16)
    width = tensors["a.right.lam"].numel()
    tensors["a.right.lam"] = torch.linspace(-9.0, 1.0, width).to(torch.bfloat16)  # decays from almost one to almost zero
    tensors["a.right.conv"] = (tensors["a.right.conv"].float() * 4.0).to(torch.bfloat16)
    for name in ("a.right.x.b", "a.right.y.b", "a.right.conv.b", "a.right.ra.b", "a.right.ri.b"):
        tensors[name] = (tensors[name].float() * 4.0).to(torch.bfloat16)
    return tensors


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", RECURRENCE_CASES, ids=lambda c: "x".join(map(str, c)))
def test_linear_recurrence_whole_in_portions_and_one_by_one(dtype, case):
    """The convolution's kept rows (their bias included) and the state carry from step to step, start at zero in a slot
    that an earlier request used, and every cut of the rows gives the plain result."""
    from part_helpers import Session, load_part

    part, raw = _recurrence_part(case)
    w = {k: v.double() for k, v in load_part(part, dtype, tensors=_recurrence_tensors(part, sum(case))).items()}
    tokens = 90
    x = (torch.randn((tokens, case[-1]), generator=torch.Generator().manual_seed(case[0])) * 1.5).to(dtype)
    expected = plain.linear_recurrence(x.double(), w, raw, "a.right.")
    session = Session([part.cache_need()], dtype, page_size=4, num_pages=4, num_slots=1)
    for cuts in CUTS(tokens):
        close(dtype, _run_part(part, session, x, cuts), expected, f"cut as {cuts[:4]}...")
    # the state and the decays matter at this bound: without memory between tokens the rows are others
    forgetful = {**w, "a.right.lam": torch.full_like(w["a.right.lam"], 30.0), "a.right.ra.b": torch.full_like(w["a.right.ra.b"], 9.0)}
    assert float((plain.linear_recurrence(x.double(), forgetful, raw, "a.right.") - expected).abs().max()) > 3 * tolerance(dtype, expected.numpy())


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_linear_recurrence_over_a_long_prompt_and_long_decoding(dtype):
    from part_helpers import Session, load_part

    part, raw = _recurrence_part((128, 2, 4, 48))
    w = {k: v.double() for k, v in load_part(part, dtype, tensors=_recurrence_tensors(part, 3)).items()}
    x = (torch.randn((700, 48), generator=torch.Generator().manual_seed(6)) * 1.5).to(dtype)
    expected = plain.linear_recurrence(x.double(), w, raw, "a.right.")
    session = Session([part.cache_need()], dtype, page_size=4, num_pages=4, num_slots=1)
    for cuts in ([700], [300] + [1] * 400, [3, 260, 257, 180]):
        close(dtype, _run_part(part, session, x, cuts), expected, f"cut as {cuts[:3]}...")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [(512, 2, 4, 48), (66, 2, 3, 40), (36, 6, 1, 24), (300, 1, 6, 32)], ids=lambda c: "x".join(map(str, c)))
def test_linear_recurrence_steps_of_many_requests(dtype, case):
    """Nineteen requests with prompts of 1 to 19 tokens, then five steps of one token each (one kernel for all of them, in
    groups of requests), then three of them alone."""
    from part_helpers import Session, load_part

    part, raw = _recurrence_part(case)
    w = {k: v.double() for k, v in load_part(part, dtype, tensors=_recurrence_tensors(part, sum(case))).items()}
    g = torch.Generator().manual_seed(case[0])
    xs = {f"r{i}": (torch.randn((i + 1 + (8 if i % 7 == 0 else 5), case[-1]), generator=g) * 1.5).to(dtype) for i in range(19)}
    steps = [[(name, int(name[1:]) + 1) for name in xs]] + [[(name, 1) for name in xs]] * 5
    steps += [[(name, 1) for name in ("r0", "r7", "r14")]] * 3
    session = Session([part.cache_need()], dtype, page_size=4, num_pages=4, num_slots=19)
    got = _run_together(part, session, xs, steps)
    for name, x in xs.items():
        close(dtype, got[name], plain.linear_recurrence(x.double(), w, raw, "a.right."), name)


# ---- two mixers side by side, added with constants ---------------------------------------------------------------------------
PAIR_CASES = [(sink(4, 2, 16, 0.7, 8, 3), recurrence(48, 3, 4), 0.8, 1.3, 64, 4), (sink(6, 1, 12, 0.9, 5, 7), recurrence(54, 9, 1), -0.7, 1.9, 100, 8),
              (sink(3, 3, 10, 1.1, 11, 1), recurrence(40, 1, 5), 1.0, 1.0, 30, 2), (sink(2, 1, 72, 0.3, 20, 2), recurrence(64, 2, 2), 2.5, 0.25, 40, 16)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", PAIR_CASES, ids=["a", "b", "c", "d"])
def test_pair_alone_and_in_batches_of_unequal_requests(dtype, case):
    """Five unequal requests, at most two at a time on two state slots and a pool that holds two requests' pages: portions
    of one beside single tokens of another, each equal to the request alone."""
    from part_helpers import Session, load_part

    left, right, ls, rs, width, page = case
    part, raw = _mixer(parallel(left, right, ls, rs), width)
    assert part.fused
    w = {k: v.double() for k, v in load_part(part, dtype, seed=width).items()}
    xs = _unequal_rows(width, page, dtype)
    expected = {name: plain.parallel_mixer(x.double(), w, raw, "a.", 1e-5) for name, x in xs.items()}
    for key in ("left_scale", "right_scale"):  # each constant shows in 32-bit
        other = plain.parallel_mixer(xs["p"].double(), w, {**raw, key: raw[key] * 1.05}, "a.", 1e-5)
        assert float((other - expected["p"]).abs().max()) > 3 * tolerance("float32", expected["p"].numpy())
    session = Session(_needs(part), dtype, page_size=page, num_pages=-(-70 // page) - (-48 // page), num_slots=2)
    close(dtype, _run_part(part, session, xs["p"], [70]), expected["p"], "alone, whole")
    got = _run_together(part, session, xs, UNEQUAL)
    for name in xs:
        close(dtype, got[name], expected[name], f"request {name} in batches")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_pair_of_sides_that_keep_their_own_products(dtype):
    """A left side that cannot leave its outer products to the pair (no gate): both sides run whole and a kernel adds."""
    from part_helpers import Session, load_part
    from kirai_b200.parts import GatedLinearRecurrence, GQAttention, ScaledPairMixer

    left = GQAttention("a.left.", 40, 4, 2, 16, None, names={"q": "q", "k": "k", "v": "v", "o": "o"}, out_dtype=torch.float32)
    right = GatedLinearRecurrence("a.right.", 40, 32, 2, 3, out_dtype=torch.float32)
    part = ScaledPairMixer(left, right, 40, 0.6, -1.2, out_dtype=torch.float32)
    assert not part.fused
    w = {k: v.double() for k, v in load_part(part, dtype, seed=8).items()}
    x = torch.randn((60, 40), generator=torch.Generator().manual_seed(2)).to(dtype)
    n = x.double()
    q, k, v = ((n @ w[f"a.left.{name}"].T).view(60, -1, 16) for name in "qkv")
    see = plain.causal(60)
    heads = [torch.softmax((q[:, h] @ k[:, h // 2].T * 0.25).masked_fill(~see, float("-inf")), -1) @ v[:, h // 2] for h in range(4)]
    expected = 0.6 * (torch.cat(heads, -1) @ w["a.left.o"].T) - 1.2 * plain.linear_recurrence(n, w, recurrence(32, 2, 3), "a.right.")
    session = Session(_needs(part), dtype, page_size=4, num_pages=16, num_slots=1)
    for cuts in ([60], [20, 2, 38], [50] + [1] * 10):
        close(dtype, _run_part(part, session, x, cuts), expected, f"cut as {cuts[:3]}")


# ---- the feed-forward, the embedding --------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff", [(64, 96), (100, 33), (48, 40), (512, 256)])
def test_clamped_feed_forward(dtype, width, ff):
    """Steps of few and of many rows (the weight-streaming and the persistent product), limits that bind on both sides of
    the up rows and on top of the gate rows only."""
    from part_helpers import DEV, load_part
    from kirai_b200.parts import GatedMLP

    for limit in (0.7, 3.0):
        part = GatedMLP("m.", width, ff, "clamped", names={"gate": "gate", "up": "up", "down": "down"}, out_dtype=torch.float32, limit=limit,
                        slope=1.702)
        w = {k: v.double() for k, v in load_part(part, dtype, seed=width).items()}
        x = (torch.randn((400, width), generator=torch.Generator().manual_seed(ff)) * 3.0).to(dtype)
        expected = plain.clamped_ffn(x.double(), w, {"limit": limit}, "m.")
        loose = plain.clamped_ffn(x.double(), w, {"limit": limit * 1.2}, "m.")
        assert float((loose - expected).abs().max()) > 3 * tolerance(dtype, expected.numpy())
        for rows in (1, 5, 17, 100, 200, 400):
            got = part.forward(x[:rows].to(DEV), None).cpu()
            assert got.dtype == torch.float32
            assert float((got.double() - expected[:rows]).abs().max()) <= tolerance(dtype, expected.numpy()), rows
    with pytest.raises(ValueError):
        GatedMLP("m.", width, ff, "clamped")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_with_a_learned_position_table(dtype):
    from part_helpers import DEV, load_part
    from kirai_b200.csrc import ops
    from kirai_b200.parts import Embedding

    for width, scale in ((64, 1.0), (37, 2.5)):
        part = Embedding("e", 20, width, scale=scale, position_table=("p", 50))
        w = load_part(part, dtype, seed=width)
        ids, positions = torch.tensor([3, 0, 19, 3, 7], dtype=torch.int32), torch.tensor([0, 49, 7, 31, 1], dtype=torch.int32)
        got = part.forward(ids.to(DEV), positions.to(DEV)).cpu()
        assert torch.allclose(got, w["e"][ids.long()] * scale + w["p"][positions.long()], rtol=1e-6, atol=1e-7)
        part.forward(ids.to(DEV), (positions + 1).to(DEV))  # one position beyond the table: reported, not read
        with pytest.raises(ops.KernelError):
            ops.check_device_errors(torch.device(DEV))


# --------------------------------------------------------------------------- whole models (GPU)
def check(dtype, got, reference, rows, what):
    expected = np.asarray(reference)[rows]
    assert got.shape == expected.shape, what
    diff = float(np.abs(got - expected).max())
    assert diff <= tolerance(dtype, reference), f"{what}: max abs diff {diff} (bound {tolerance(dtype, reference)})"


@pytest.fixture(scope="module", params=["A", "B", "C"])
def tiny(request, tmp_path_factory):
    raw, page, seed = TINY[request.param]
    folder = str(tmp_path_factory.mktemp(f"fosavik{request.param}"))
    write_model(folder, raw, seed)
    config, weights = read_model_folder(folder)
    assert config == raw
    sequences = {rid: random_tokens(n, raw["vocab"], 300 + k)
                 for k, (rid, n) in enumerate([("a", 75), ("b", 40), ("c", 53), ("d", 9), ("e", 61), ("f", 34)])}
    reference = {rid: plain.forward(config, weights, toks).numpy() for rid, toks in sequences.items()}
    return dict(name=request.param, folder=folder, raw=raw, config=config, weights=weights, page=page,
                sequences=sequences, reference=reference)


@pytest.mark.gpu
def test_stream_copies_sum_after_every_layer(tiny):
    """In 32-bit the copies' sum after each layer equals the plain one."""
    from kirai_b200.engine.batch import StepEntry
    from kirai_b200.engine.runner import ModelRunner
    from kirai_b200.parts.block import Block

    runner = ModelRunner.from_folder(tiny["folder"], dtype="float32", page_size=tiny["page"], max_tokens=128, num_slots=2)
    tokens = tiny["sequences"]["b"]
    _, streams = plain.forward(tiny["config"], tiny["weights"], tokens, return_layers=True)
    kept, original = [], Block.forward

    def recording(self, resid, *args, **kwargs):
        streams, left = original(self, resid, *args, **kwargs)
        copies = left.mix.shape[0]
        xs = (streams if streams.dim() == 3 else streams[:, None].expand(-1, copies, -1)).double()
        kept.append((torch.einsum("tfw,fg->tw", xs, left.mix.double()) + left.add.double().sum() * left.rows.double()).cpu())
        return streams, left

    Block.forward = recording
    try:
        runner.step([StepEntry(runner.cache.open("b"), tokens, [0])])
    finally:
        Block.forward = original
    assert len(kept) == len(streams)
    for index, total in enumerate(kept):
        assert float((total - streams[index]).abs().max()) < 2e-4 * max(1.0, float(streams[index].abs().max())), f"after layer {index}"


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_then_last_tokens_one_by_one(tiny, dtype, tmp_path):
    from replay_client import Replay

    replay = Replay(tiny["folder"], dtype, str(tmp_path / "out"), max_tokens=160, page_size=tiny["page"])
    for rid in ("a", "d"):
        toks = tiny["sequences"][rid]
        got = replay.step([(rid, toks, range(len(toks)))], end=[rid])
        check(dtype, got, tiny["reference"][rid], list(range(len(toks))), f"whole {rid}")
    for rid in ("a", "c"):
        toks = tiny["sequences"][rid]
        head = len(toks) - 32
        got = replay.step([(rid, toks[:head], [head - 1])])
        check(dtype, got, tiny["reference"][rid], [head - 1], f"{rid} prompt")
        for i in range(head, len(toks)):
            got = replay.step([(rid, [toks[i]], [0])], end=[rid] if i == len(toks) - 1 else [])
            check(dtype, got, tiny["reference"][rid], [i], f"{rid} decode at {i}")
    assert replay.close() == 0


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_whole_and_in_portions(tiny, dtype, tmp_path):
    """A prompt long enough for the recurrences' products and chunks of many tokens, whole and beside a second request;
    the same prompt in portions; both against the plain model."""
    from replay_client import Replay

    toks = random_tokens(330, tiny["raw"]["vocab"], 77)
    other = tiny["sequences"]["d"]
    reference = plain.forward(tiny["config"], tiny["weights"], toks).numpy()
    rows = [0, 1, 63, 64, 65, 127, 128, 200, 255, 256, 257, 300, 328, 329]
    replay = Replay(tiny["folder"], dtype, str(tmp_path / "out"), max_tokens=512, page_size=tiny["page"])
    got = replay.step([("long", toks, rows), ("d", other, [len(other) - 1])], end=["long", "d"])
    check(dtype, got[: len(rows)], reference, rows, "whole, beside a short request")
    check(dtype, got[len(rows) :], tiny["reference"]["d"], [len(other) - 1], "the short request beside it")
    done = 0
    for size in (30, 3, 260, 1, 10, 26):
        want = [r - done for r in rows if done <= r < done + size]
        got = replay.step([("again", toks[done : done + size], want)], end=["again"] if done + size == len(toks) else [])
        if want:
            check(dtype, got, reference, [r + done for r in want], f"portion at {done}")
        done += size
    assert done == len(toks) and replay.close() == 0


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_down_to_two_tokens(tiny, dtype, tmp_path):
    """Portions that end inside a page, inside a window, among the kept first keys and inside the convolution's reach."""
    from replay_client import Replay

    replay = Replay(tiny["folder"], dtype, str(tmp_path / "out"), max_tokens=96, page_size=tiny["page"])
    toks = tiny["sequences"]["a"]
    for sizes in ([13, 2, 7, 16, 5, 3, 2, 11, 9, 2, 5], [2] * 37 + [1], [64, 11], [1, 1, 2, 3, 68]):
        assert sum(sizes) == len(toks)
        start = 0
        for size in sizes:
            got = replay.step([("a", toks[start : start + size], range(size))])
            check(dtype, got, tiny["reference"]["a"], list(range(start, start + size)), f"portion at {start}+{size}")
            start += size
        replay.step([], end=["a"])
    assert replay.close() == 0


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_on_a_pool_that_runs_full(tiny, dtype, tmp_path):
    """Six unequal requests, at most four live on four state slots, portions of some beside single tokens of others, on
    a pool exactly as large as the most that live requests hold at once: later requests get pages and slots that
    earlier ones gave back, and every logit equals what the request gives alone."""
    from replay_client import Replay
    from test_replay import mixed_schedule, tokens_held_at_most

    sequences, reference, page = tiny["sequences"], tiny["reference"], tiny["page"]
    steps = mixed_schedule(sequences)
    most = tokens_held_at_most(steps, page)
    replay = Replay(tiny["folder"], dtype, str(tmp_path / "out"), max_tokens=most, page_size=page,
                    extra=("--stats", str(tmp_path / "out" / "stats.json"), "--max-requests", "4"))
    for entries, end in steps:
        batch = [(rid, sequences[rid][first : first + count], range(count)) for rid, first, count in entries]
        got = replay.step(batch, end=end)
        row = 0
        for rid, first, count in entries:
            check(dtype, got[row : row + count], reference[rid], list(range(first, first + count)), f"mixed {rid} at {first}+{count}")
            row += count
    assert replay.close() == 0
    stats = replay.stats()
    assert stats["live_requests"] == 0
    for group in stats["groups"]:
        assert group["used"] == 0 and group["handed_out"] > group["pages"] == most // page


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_and_long_decoding(tiny, dtype, tmp_path):
    """330 tokens one by one from the first: the kept keys fill up, the windows pass over them, the states run long."""
    from replay_client import Replay

    toks = random_tokens(330, tiny["raw"]["vocab"], 17)
    reference = plain.forward(tiny["config"], tiny["weights"], toks).numpy()
    replay = Replay(tiny["folder"], dtype, str(tmp_path / "out"), max_tokens=352, page_size=tiny["page"])
    for i, token in enumerate(toks):
        got = replay.step([("long", [token], [0])])
        check(dtype, got, reference, [i], f"decode at {i}")
    assert replay.close() == 0


@pytest.mark.gpu
def test_positions_beyond_the_table_are_refused(tiny):
    from kirai_b200.engine.batch import StepEntry
    from kirai_b200.engine.runner import ModelRunner
    from kirai_b200.engine.step import StepError

    limit = tiny["raw"]["max_positions"]
    runner = ModelRunner.from_folder(tiny["folder"], dtype="bfloat16", page_size=tiny["page"], max_tokens=limit + 64, num_slots=1)
    request = runner.cache.open("r")
    logits = runner.step([StepEntry(request, random_tokens(limit, tiny["raw"]["vocab"], 1), [limit - 1])])
    assert bool(torch.isfinite(logits).all())
    with pytest.raises(StepError):
        runner.step([StepEntry(request, [1], [0])])


def test_bounds_would_show_a_fault_in_each_mechanism(tiny):
    """What each of these faults costs a whole model's logits, against the bfloat16 bound of its tests."""
    tokens, true = tiny["sequences"]["a"], tiny["reference"]["a"]
    bound = tolerance("bfloat16", true)

    def with_patched(name, replacement):
        original = getattr(plain, name)
        setattr(plain, name, replacement(original))
        try:
            return plain.forward(tiny["config"], tiny["weights"], tokens).numpy()
        finally:
            setattr(plain, name, original)

    faults = {
        "no sink": with_patched("softmax_with_sink", lambda f: lambda s: torch.softmax(s, dim=-1)),
        "mix transposed": with_patched("streams_update", lambda f: lambda xs, y, w, p: f(xs, y, {**w, p + "mix": w[p + "mix"].T}, p)),
        "first map only": with_patched("map_weight", lambda f: lambda *a: 0.0 * f(*a)),
        "no position vectors": with_patched("embedded", lambda f: lambda w, t: w["embed"][torch.tensor(t)]),
        "no limit": with_patched("clamped_ffn", lambda f: lambda n, w, mlp, p: f(n, w, {**mlp, "limit": 1e6}, p)),
        "no state": with_patched("linear_recurrence", lambda f: lambda n, w, m, p: torch.cat([f(n[t : t + 1], w, m, p) for t in range(n.shape[0])])),
    }
    for name, other in faults.items():
        if name == "mix transposed" and tiny["raw"]["streams"] == 1:
            continue
        if name == "no limit" and tiny["name"] == "C":
            continue  # (its limits are wide)
        assert float(np.abs(other - true).max()) > bound, name


def _sure_tokens(config, weights, prompt, generated):
    """How many of the generated tokens, from the first on, are chosen by a margin that rounding to bfloat16 cannot close."""
    logits = plain.forward(config, weights, list(prompt) + list(generated))
    top2 = torch.topk(logits[len(prompt) - 1 : -1], 2, dim=-1).values
    sure = ((top2[:, 0] - top2[:, 1]) > 0.03 * float(logits.abs().max())).tolist()
    return sure.index(False) if False in sure else len(sure)


def _plain_greedy(config, weights, prompt, count):
    tokens = list(prompt)
    for _ in range(count):
        logits = plain.forward(config, weights, tokens)[-1]
        tokens.append(int(torch.nonzero(logits == logits.max())[0]))
    return tokens[len(prompt):]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(tiny, dtype):
    """Five prompts through the scheduler (three at a time on three state slots, prompts in portions of 16, decode steps
    from captured graphs) give the plain implementation's greedy tokens."""
    from kirai_b200 import Engine, SamplingParams

    engine = Engine(tiny["folder"], dtype=dtype, page_size=tiny["page"], max_prefill_tokens=16, max_concurrent_requests=3,
                    max_new_tokens=16, max_cache_tokens=256)
    prompts = [random_tokens(n, tiny["raw"]["vocab"], 50 + n) for n in (5, 11, 17, 3, 24)]
    outputs = engine.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=8))
    compared = 0
    for prompt, output in zip(prompts, outputs):
        expected = _plain_greedy(tiny["config"], tiny["weights"], prompt, 8)
        assert output.finish_reason == "length" and (output.prompt_tokens, output.completion_tokens) == (len(prompt), 8)
        count = 8 if dtype == "float32" else _sure_tokens(tiny["config"], tiny["weights"], prompt, expected)
        assert output.token_ids[:count] == expected[:count]
        compared += count
    assert compared >= (40 if dtype == "float32" else 6)
    stats = engine.stats()
    assert engine.counters["graph_steps"] > 0
    assert stats["cache"]["live_requests"] == 0 and all(g["used"] == 0 for g in stats["cache"]["groups"])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_captured_decode_steps_give_the_step_functions_logits(tiny, dtype):
    """The captured step and the step queued behind it on requests of unequal lengths, against the step function on twins
    of those requests (a step advances the states, so it cannot run twice on the same ones)."""
    from kirai_b200 import Engine
    from kirai_b200.engine.batch import StepEntry

    engine = Engine(tiny["folder"], dtype=dtype, page_size=tiny["page"], max_prefill_tokens=64, max_concurrent_requests=6,
                    max_new_tokens=16, max_cache_tokens=512)
    runner, vocab, lens = engine.runner, tiny["raw"]["vocab"], (60, 3, 21)
    cache = runner.cache
    requests, twins = ([cache.open((kind, i)) for i in range(3)] for kind in ("captured", "eager"))
    for group in (requests, twins):
        for request, n in zip(group, lens):
            runner.step([StepEntry(request, random_tokens(n, vocab, n), [])])
    assert all(cache.reserve(request, 2) for request in requests)
    tables = [cache.block_table_array(requests, g) for g in range(len(cache.groups))]
    graph, fresh = engine.graphs.get(3, max(t.shape[1] for t in tables), [n + 1 for n in lens])
    tokens, greedy = random_tokens(3, vocab, 5), ([0.0] * 3, [1.0] * 3, [0.0] * 3)
    graph.load_inputs(tokens, list(lens), [r.slot for r in requests], tables, *greedy)
    assert fresh
    graph.capture()
    first = graph.launch()
    captured = [graph.logits_out[:3].clone()]
    graph.load_inputs(None, [n + 1 for n in lens], [r.slot for r in requests], tables, *greedy)
    second = graph.launch()
    captured.append(graph.logits_out[:3].clone())
    sampled = first.wait()
    second.wait()
    for got, ids in zip(captured, (tokens, sampled)):
        eager = runner.step([StepEntry(r, [int(t)], [0]) for r, t in zip(twins, ids)])
        close(torch.float32 if dtype == "float32" else torch.bfloat16, got.cpu(), eager.cpu(), "captured against eager")


@pytest.mark.gpu
def test_eviction_and_recompute_give_the_same_sampled_tokens(tiny):
    """Seeded temperature sampling on a pool too small for both requests: one is evicted, its pages and its state slots
    go back, and its recomputation (states from zero again) gives the tokens of the roomy run."""
    from kirai_b200 import Engine, SamplingParams

    params = SamplingParams(temperature=0.8, top_p=0.95, seed=5, max_new_tokens=14)
    prompts = [random_tokens(17, tiny["raw"]["vocab"], 1), random_tokens(18, tiny["raw"]["vocab"], 2)]
    roomy = Engine(tiny["folder"], dtype="float32", page_size=tiny["page"], max_new_tokens=16, max_cache_tokens=256)
    expected = [o.token_ids for o in roomy.generate(prompts, params)]
    tight = Engine(tiny["folder"], dtype="float32", page_size=tiny["page"], max_new_tokens=16, max_cache_tokens=48)
    outputs = tight.generate(prompts, params)
    assert [o.token_ids for o in outputs] == expected


@pytest.mark.gpu
def test_command_line_generates(tiny):
    prompt = random_tokens(9, tiny["raw"]["vocab"], 77)
    result = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "kirai"), "generate", "--snapshot", tiny["folder"],
                             "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "6", "--temperature", "0",
                             "--dtype", "float32", "--page-size", str(tiny["page"])], capture_output=True, text=True, timeout=600)
    assert result.returncode == 0, result.stderr
    expected = _plain_greedy(tiny["config"], tiny["weights"], prompt, 6)
    assert json.loads(result.stdout.strip().splitlines()[-1])["token_ids"] == expected
