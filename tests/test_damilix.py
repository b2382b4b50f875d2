"""The Damilix decoder against its plain implementation (``plain_damilix``): each mechanism alone (normed embedding rows,
latent attention with queries straight from the stream, its sinks and gates, both rotations, gated linear attention in its
three forms, the corrected softmax router with identity experts, the gated shared branch, the input of the token's own), then
whole models through trace replay (whole, decoded one by one, in portions down to two tokens, mixed batches on a pool that
runs full, long prompts, long decoding) and greedy generation through the engine and the command line.

Configurations and weights are made here.  Where random weights would hide a fault (a far key among hundreds, a sink, decays
that forget within a chunk, a state that must come back) rows or weights are scaled so that it shows."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_damilix as plain
from plain_qwen3 import read_model_folder
from tiny_configs import random_tokens

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]


def rot(base, dims, scaling=None):
    out = {"base": base, "dims": dims}
    if scaling:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def latent(kind, heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, scaling=None):
    return {"type": kind, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                                    "rot": rot(base, rot_dim, scaling)}}


def gla(heads, dim, vdim, tau):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, scale, identity=0, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if identity:
        out["router"]["identity"] = identity
    if shared:
        out["shared"] = {"ff": shared}
    return out


def layer(entry, mlp):
    return {**entry, "mlp": mlp}


NEIGHBOURS, HALVES = "latent_attention", "latent_attention_2"

# A: sizes in multiples of 8, every kind of mixer and feed-forward, a layer without feed-forward.  B: nothing a multiple of 8,
# a shared branch that cannot be stacked behind the experts, more identity experts than a token uses, heads that do not divide
# the attention kernels' tiles, stretched frequencies that reach the clamp on both sides.  C: sizes and
# counts of one (one head, one expert a token, tau 1, no identity expert, no shared branch), a latent narrower than a head.
CONFIG_A = {
    "architecture": "Damilix", "width": 64, "vocab": 200, "norm": {"eps": 1e-5}, "token_side": {"dim": 8},
    "layers": [
        layer(latent(NEIGHBOURS, 4, 16, 8, 24, 32, 0.6, base=300.0, scaling=(4.0, 32, 8.0, 1.0)), dense(96)),
        layer(gla(2, 24, 16, 8.0), moe(16, 8, 3, 1.7, identity=2, shared=24)),
        layer(latent(HALVES, 2, 24, 16, 8, 24, 0.5), None),
        layer(gla(4, 8, 32, 3.0), dense(40)),
        layer(latent(HALVES, 8, 8, 8, 16, 40, 0.7, base=500.0), moe(24, 6, 2, 2.2, identity=1, shared=40)),
    ],
}
CONFIG_B = {
    "architecture": "Damilix", "width": 100, "vocab": 131, "norm": {"eps": 1e-3}, "token_side": {"dim": 5},
    "layers": [
        layer(gla(3, 20, 12, 2.0), moe(12, 5, 2, 0.8, identity=3, shared=21)),
        layer(latent(HALVES, 5, 10, 6, 12, 18, 0.7, base=50.0), dense(33)),
        layer(latent(NEIGHBOURS, 3, 12, 10, 20, 22, 0.6, base=77.0, scaling=(2.0, 16, 4.0, 0.5)), moe(20, 4, 3, 1.4, shared=12)),
        layer(gla(2, 14, 37, 16.0), None),
    ],
}
CONFIG_C = {
    "architecture": "Damilix", "width": 48, "vocab": 90, "norm": {"eps": 1e-6}, "token_side": {"dim": 16},
    "layers": [layer(latent(NEIGHBOURS, 1, 32, 16, 40, 16, 0.5), moe(32, 3, 1, 1.0)), layer(gla(1, 70, 14, 1.0), moe(8, 2, 2, 1.2, identity=1))],
}
TINY = {"A": (CONFIG_A, 4, 253), "B": (CONFIG_B, 8, 151), "C": (CONFIG_C, 16, 50)}  # name -> (config, page size, seed)


def loud(tensors, raw):
    """Random weights made so that each mechanism shows: sinks of the size of large scores, biases and projections of the decays
    that spread them from forgetting at once to keeping for hundreds of tokens, routers whose scores lie far apart, corrections
    that change choices."""
    for name, t in list(tensors.items()):
        if name.endswith(".sink"):
            tensors[name] = (t.float().abs() * 12.0 + 2.0).to(torch.bfloat16)
        elif name.endswith(".a2.b"):
            tensors[name] = (t.float() * 25.0 + 2.0).to(torch.bfloat16)
        elif name.endswith((".a1", ".a2", ".router")):
            tensors[name] = (t.float() * 3.0).to(torch.bfloat16)
        elif name.endswith((".mix.g", ".side.gate", ".shared.sg")):
            tensors[name] = (t.float() * 2.0).to(torch.bfloat16)
    return tensors


def write_model(folder, raw, seed, std=0.07):
    import kirai_b200  # noqa: F401
    from kirai_b200.registry import config_from_dict, plan_for_config
    from kirai_b200.weights.random_init import random_tensors
    from kirai_b200.weights.safetensors_io import write_safetensors

    cfg = config_from_dict(raw)
    tensors = loud(random_tensors(plan_for_config(cfg).weight_specs(), seed, std=std, norm_jitter=0.3, dtype=torch.bfloat16), raw)
    # (the rank between the decays' two matrices is the tensors' own: another one in the second linear layer)
    second = [i for i, entry in enumerate(raw["layers"]) if entry["type"] == "gla"][-1]
    a1, a2 = f"l{second}.mix.a1", f"l{second}.mix.a2"
    tensors[a1], tensors[a2] = tensors[a1][:7].contiguous(), tensors[a2][:, :7].contiguous()
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as handle:
        json.dump(cfg.to_dict(), handle, indent=2)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors, metadata={"format": "pt"})


def tolerance(dtype, reference):
    dtype = {torch.float32: "float32", torch.bfloat16: "bfloat16"}.get(dtype, dtype)
    peak = float(np.abs(np.asarray(reference)).max())
    return 3e-5 * max(1.0, peak) if dtype == "float32" else 0.05 * peak


def close(dtype, got, expected, what):
    got, expected = np.asarray(got, dtype=np.float64), np.asarray(expected, dtype=np.float64)
    assert got.shape == expected.shape, what
    if got.size:
        worst = float(np.abs(got - expected).max())
        assert worst <= tolerance(dtype, expected), f"{what}: max abs diff {worst} (bound {tolerance(dtype, expected)})"


# --------------------------------------------------------------------------- no GPU
def test_config_reads_every_size_and_round_trips():
    import kirai_b200  # noqa: F401
    from kirai_b200.config.base import ConfigError
    from kirai_b200.parts.base import KVCacheNeed
    from kirai_b200.registry import config_from_dict, plan_for_config

    for raw in (CONFIG_A, CONFIG_B, CONFIG_C):
        cfg = config_from_dict(raw)
        assert cfg.to_dict() == raw and config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
        plan = plan_for_config(cfg)
        assert plan.capture_safe() and plan.kernels_only()
        specs = plan.weight_specs()
        assert specs["side.embed"].shape == (raw["vocab"], len(raw["layers"]) * raw["token_side"]["dim"])
        for i, entry in enumerate(raw["layers"]):
            m, need, mlp = entry["mixer"], plan.cache_needs[i], entry["mlp"]
            if entry["type"] == "gla":
                assert need.shape == (m["heads"] * m["dim"] * m["vdim"],) and need.dtype == torch.float32
            else:
                assert isinstance(need, KVCacheNeed) and (need.kv_heads, need.key_dim, need.value_dim) == (1, m["kv_rank"] + m["rot_dim"], m["kv_rank"])
            assert (f"l{i}.norm2" in specs) == (mlp is not None) and f"l{i}.side.norm" in specs
            if mlp is not None and mlp["kind"] == "moe":
                outputs = mlp["router"]["experts"] + mlp["router"].get("identity", 0)
                assert specs[f"l{i}.mlp.router"].shape == (outputs, raw["width"]) and specs[f"l{i}.mlp.correction"].shape == (outputs,)
                assert (f"l{i}.mlp.shared.sg" in specs) == ("shared" in mlp) and f"l{i}.mlp.e{mlp['router']['experts']}.up" not in specs
    for change in (lambda r: r["layers"][0].update(type="attention"),
                   lambda r: r["layers"][0]["mixer"]["rot"].update(dims=6),
                   lambda r: r["layers"][0]["mixer"].pop("scale"),
                   lambda r: r["layers"][1]["mixer"].update(tau=0.0),
                   lambda r: r["layers"][1]["mlp"]["router"].update(top=11),
                   lambda r: r["layers"][1]["mlp"]["router"].pop("scale"),
                   lambda r: r["layers"][1]["mlp"].update(kind="gated"),
                   lambda r: r.pop("token_side"),
                   lambda r: r["norm"].update(eps=-1.0)):
        bad = json.loads(json.dumps(CONFIG_A))
        change(bad)
        with pytest.raises(ConfigError):
            config_from_dict(bad)


def test_sizes_that_only_the_tensors_give():
    """The rank of the decays' projection is read from the stored tensors; both of a layer's must agree."""
    import kirai_b200  # noqa: F401
    from kirai_b200.parts import DecayedLinearAttention
    from kirai_b200.weights.loader import WeightError, from_tensors
    from kirai_b200.weights.random_init import random_tensors

    specs = DecayedLinearAttention("m.", 12, 2, 3, 4, 2.0, 1e-5).weight_specs()
    tensors = random_tensors(specs, 0)
    assert tensors["m.a1"].shape == (16, 12) and tensors["m.a2"].shape == (6, 16)
    from_tensors(tensors, specs, "cpu")
    other = {**tensors, "m.a1": torch.zeros((5, 12)), "m.a2": torch.zeros((6, 5))}
    assert from_tensors(other, specs, "cpu").stored("m.a1").shape == (5, 12)
    for bad in ({**other, "m.a2": torch.zeros((6, 4))}, {**other, "m.a1": torch.zeros((5, 11))}, {**other, "m.a1": torch.zeros(5)},
                {**other, "m.a1": torch.zeros((0, 12))}):
        with pytest.raises(WeightError):
            from_tensors(bad, specs, "cpu")


def test_plain_forms_worked_by_hand():
    one = torch.ones((1, 2), dtype=torch.float64)
    # softmax shares 0.5, 0.3, 0.2; the correction lifts the last over the second; the weights are the shares, brought to 3
    w = {"m.router": torch.log(torch.tensor([[0.5, 1.0], [0.3, 1.0], [0.2, 1.0]], dtype=torch.float64)),
         "m.correction": torch.tensor([0.0, -0.1, 0.05], dtype=torch.float64)}
    ids, weights = plain.router_choice(torch.tensor([[1.0, 0.0]], dtype=torch.float64), w, moe(4, 2, 2, 3.0, identity=1), "m.")
    assert ids.tolist() == [[0, 2]] and torch.allclose(weights, torch.tensor([[15.0 / 7.0, 6.0 / 7.0]], dtype=torch.float64))
    # a sink of the score's own height takes half of a single key's weight
    p = plain.sink_softmax(one[:, :1] * 2.0, torch.ones((1, 1), dtype=torch.bool), torch.tensor(2.0, dtype=torch.float64))
    assert abs(float(p) - 0.5) < 1e-12
    # two tokens through one state cell: S = 2, then 0.5 * 2 + 3 * 1
    q, k = torch.tensor([1.0, 10.0], dtype=torch.float64).view(2, 1, 1), torch.tensor([1.0, 3.0], dtype=torch.float64).view(2, 1, 1)
    v, g = torch.tensor([2.0, 1.0], dtype=torch.float64).view(2, 1, 1), torch.log(torch.tensor([0.9, 0.5], dtype=torch.float64)).view(2, 1, 1)
    o, S = plain.linear_recurrence(q, k, v, g)
    assert torch.allclose(o.view(-1), torch.tensor([2.0, 40.0], dtype=torch.float64)) and abs(float(S) - 4.0) < 1e-12
    # the pairs of the two rotations
    x = torch.arange(1.0, 5.0, dtype=torch.float64).view(1, 1, 4)
    angles = torch.tensor([3.0, 3.0 * np.float64(np.float32(0.1))], dtype=torch.float64)
    c, s = angles.cos(), angles.sin()
    pos = torch.tensor([3])
    near = plain.rotate(x, pos, rot(100.0, 4), True).view(-1)
    half = plain.rotate(x, pos, rot(100.0, 4), False).view(-1)
    assert torch.allclose(near, torch.stack([c[0] - 2 * s[0], 2 * c[0] + s[0], 3 * c[1] - 4 * s[1], 4 * c[1] + 3 * s[1]]), atol=1e-6)
    assert torch.allclose(half, torch.stack([c[0] - 3 * s[0], 2 * c[1] - 4 * s[1], 3 * c[0] + s[0], 4 * c[1] + 2 * s[1]]), atol=1e-6)


# ------------------------------------------------------------------ mechanisms alone
def _mixer(entry, width, eps=1e-5):
    import kirai_b200  # noqa: F401
    from kirai_b200.config.damilix import DamilixConfig
    from kirai_b200.models.damilix import mixer_for_layer

    raw = {"architecture": "Damilix", "width": width, "vocab": 16, "norm": {"eps": eps}, "token_side": {"dim": 4}, "layers": [layer(entry, None)]}
    cfg = DamilixConfig.from_dict(raw)
    return mixer_for_layer(cfg, cfg.layers[0], "a."), raw["layers"][0]["mixer"]


def _loaded(part, dtype, seed, std=0.1, change=None):
    """The part with loud random weights; returns them in 64-bit."""
    from kirai_b200.weights.random_init import random_tensors
    from part_helpers import load_part

    renamed = {name.replace("a.", "a.mix.", 1): t for name, t in random_tensors(part.weight_specs(), seed, std=std, norm_jitter=0.3).items()}
    tensors = {name.replace("a.mix.", "a.", 1): t for name, t in loud(renamed, None).items()}
    if change is not None:
        change(tensors)
    return {name: t.double() for name, t in load_part(part, dtype, tensors=tensors).items()}


def _run_together(part, session, xs, steps):
    """The part's output rows for several requests (``xs``: name -> rows [T, width]) under a schedule: ``steps`` is a
    list of steps, each a list of (name, count) that run as one batch.  A request is closed after its last row."""
    names, offset, table = list(xs), {}, []
    for name in names:
        offset[name] = sum(t.shape[0] for t in table)
        table.append(xs[name])
    table = torch.cat(table)
    done, out = {name: 0 for name in names}, None
    for step in steps:
        batch = session.batch([(name, list(range(offset[name] + done[name], offset[name] + done[name] + count))) for name, count in step])
        rows = batch.token_ids.cpu().long()
        y = part.forward(table[rows].cuda(), batch, session.cache.layer_view(0)).float().cpu()
        out = torch.zeros((table.shape[0], y.shape[1])) if out is None else out
        out[rows] = y
        session.commit()
        for name, count in step:
            done[name] += count
            if done[name] == xs[name].shape[0]:
                session.cache.close(session.requests.pop(name))
    assert all(done[name] == xs[name].shape[0] for name in names)
    return {name: out[offset[name] : offset[name] + xs[name].shape[0]] for name in names}


def _run_part(part, session, x, cuts):
    return _run_together(part, session, {"s": x}, [[("s", size)] for size in cuts])["s"]


def CUTS(n):
    return [n], [37, 2, 19, 1, 1, 3, n - 63], [n - 10] + [1] * 10, [2] * (n // 2) + [1] * (n % 2), [1] * n


UNEQUAL = [[("p", 40), ("q", 2)], [("p", 1), ("q", 20)], [("p", 1), ("q", 1)], [("q", 10), ("p", 28)],      # p and q end here
           [("r", 7), ("s", 1)], [("r", 1), ("s", 30)], [("s", 1), ("r", 1)], [("s", 16)],                   # r ends, then s
           [("t", 1)], [("t", 1)]]


def _unequal_rows(width, seed, dtype):
    g = torch.Generator().manual_seed(seed)
    return {name: (torch.randn((n, width), generator=g) * 1.5).to(dtype) for name, n in (("p", 70), ("q", 33), ("r", 9), ("s", 48), ("t", 2))}


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 100, 7, 4096 + 24])
def test_normed_embedding_rows_and_their_copy(dtype, width):
    from part_helpers import DEV, load_part
    from kirai_b200.csrc import ops
    from kirai_b200.parts import Embedding

    part = Embedding("e", 20, width, norm=("n", 1e-3))
    w = {k: v.double() for k, v in load_part(part, dtype, seed=width).items()}
    ids = torch.tensor([3, 0, 19, 3, 7], dtype=torch.int32)
    expected = plain.unit_norm(w["e"][ids.long()], w["n"], 1e-3)
    close(torch.float32, part.forward(ids.to(DEV)).cpu(), expected, "stream")
    stream, copy = part.forward_with_copy(ids.to(DEV))
    close(torch.float32, stream.cpu(), expected, "stream beside its copy")
    assert (copy is None) == (dtype == torch.float32)
    if copy is not None:
        assert torch.equal(copy, stream.to(torch.bfloat16))
    part.forward(torch.tensor([20], dtype=torch.int32).to(DEV))  # one id beyond the table: reported, not read
    with pytest.raises(ops.KernelError):
        ops.check_device_errors(torch.device(DEV))
    with pytest.raises(ValueError):
        Embedding("e", 20, width, norm=("n", 1e-3), scale=2.0)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,dim", [(64, 8), (100, 5), (36, 24), (512, 64)])
def test_an_input_of_the_tokens_own(dtype, width, dim):
    """For each of three layers' parts of a token's row; steps of few and of many tokens.  Another layer's part, or no gate,
    is far outside the bound."""
    from types import SimpleNamespace

    from part_helpers import DEV, load_part
    from kirai_b200.parts import TokenSideInput

    g = torch.Generator().manual_seed(dim)
    x = torch.randn((300, width), generator=g) * 2.0
    ids = torch.randint(0, 30, (300,), generator=g)
    config = {"token_side": {"dim": dim}}
    for index in (0, 2):
        part = TokenSideInput("s.", "side.embed", width, dim, index * dim, 30, 3 * dim, 1e-5)
        w = {k: v.double() for k, v in load_part(part, dtype, seed=width + index).items()}
        read = x.to(dtype).double()  # what the products read; the stream itself stays 32-bit
        added = plain.token_input(read, ids, w, config, index, "s.", 1e-5)
        other = plain.token_input(read, ids, w, config, 1, "s.", 1e-5)
        assert float((added - other).abs().max()) > 5 * tolerance(dtype, added.numpy())
        for rows in (1, 5, 300):
            resid = x[:rows].to(DEV)
            copy = part.add(x[:rows].to(dtype).to(DEV), resid, SimpleNamespace(token_ids=ids[:rows].to(torch.int32).to(DEV)))
            bound = tolerance(dtype, added.numpy())
            assert float((resid.cpu().double() - x[:rows].double() - added[:rows]).abs().max()) <= bound + 1e-5, (index, rows)
            assert copy is None if dtype == torch.float32 else torch.equal(copy, resid.to(torch.bfloat16))
    with pytest.raises(ValueError):
        TokenSideInput("s.", "side.embed", width, dim, 3 * dim, 30, 3 * dim, 1e-5)


LATENT_CASES = [  # kind, heads, dim, rot_dim, vdim, kv_rank, scale, base, scaling; width, page
    ((NEIGHBOURS, 4, 16, 8, 24, 32, 0.8, 300.0, (4.0, 32, 8.0, 1.0)), 64, 4),
    ((HALVES, 6, 10, 6, 12, 18, 1.0, 50.0, None), 100, 8),
    ((NEIGHBOURS, 1, 12, 2, 20, 22, 0.7, 77.0, None), 48, 16),
    ((HALVES, 3, 24, 16, 8, 40, 0.6, 500.0, (2.0, 16, 4.0, 0.5)), 64, 4),
    ((HALVES, 16, 8, 32, 16, 96, 0.5, 10000.0, None), 72, 8),
    ((NEIGHBOURS, 20, 8, 8, 4, 200, 0.6, 900.0, (3.0, 64, 4.0, 1.0)), 56, 16),
    ((HALVES, 2, 12, 40, 16, 260, 0.5, 2000.0, None), 64, 8),  # a cached row wider than the tensor-core kernels take
]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case,width,page", LATENT_CASES, ids=lambda c: "x".join(map(str, c[1:6])) if isinstance(c, tuple) else str(c))
def test_latent_attention_whole_in_portions_and_one_by_one(dtype, case, width, page):
    """Alone in every cut, then five unequal requests on pages and slots that are used again.  Each of the mechanisms left out
    or taken the other way (sinks, gates, the pairing, the stretched frequencies' factor) is far outside the 32-bit bound."""
    from part_helpers import Session

    part, raw = _mixer(latent(*case), width)
    w = _loaded(part, dtype, width)
    xs = _unequal_rows(width, page, dtype)
    neighbours = case[0] == NEIGHBOURS
    expected = {name: plain.latent_attention(x.double(), w, raw, "a.", 1e-5, neighbours) for name, x in xs.items()}
    x = xs["p"].double()
    faults = [plain.latent_attention(x, {**w, "a.sink": w["a.sink"] - 50.0}, raw, "a.", 1e-5, neighbours),
              plain.latent_attention(x, {**w, "a.g": 0.0 * w["a.g"]}, raw, "a.", 1e-5, neighbours)]
    if raw["rot_dim"] > 2:
        faults.append(plain.latent_attention(x, w, raw, "a.", 1e-5, not neighbours))
    if case[8]:
        faults.append(plain.latent_attention(x, w, {**raw, "rot": rot(case[7], case[3])}, "a.", 1e-5, neighbours))
    for fault in faults:
        assert float((fault - expected["p"]).abs().max()) > 20 * tolerance("float32", expected["p"].numpy())
    session = Session([part.cache_need()], dtype, page_size=page, num_pages=-(-70 // page) - (-48 // page), num_slots=2)
    for cuts in CUTS(70):
        close(dtype, _run_part(part, session, xs["p"], cuts), expected["p"], f"cut as {cuts[:4]}...")
    got = _run_together(part, session, xs, UNEQUAL)
    for name in xs:
        close(dtype, got[name], expected[name], f"request {name} in batches")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", [NEIGHBOURS, HALVES])
def test_a_far_key_stands_out(dtype, kind):
    """Late tokens that repeat an early one, with queries aligned to keys: the early token takes most of the weight, hundreds
    of keys away, across page borders, in a prompt and decoded."""
    from part_helpers import Session

    heads, dim, r, vdim, rank, width, page, total = 3, 24, 8, 16, 24, 40, 8, 420
    part, raw = _mixer(latent(kind, heads, dim, r, vdim, rank, 0.35, 1e6), width)

    def align(tensors):
        # head i's unrotated query is the token's own unnormed latent through the same matrix as its key
        uk = tensors["a.uk"].float().view(heads, dim, rank)
        q = tensors["a.q"].float().view(heads, dim + r, width)
        q[:, :dim] = torch.einsum("hdk,kx->hdx", uk, tensors["a.dkv"].float()[:rank]) * 3.0
        tensors["a.q"] = q.reshape(heads * (dim + r), width).to(torch.bfloat16)

    w = _loaded(part, dtype, 5, std=0.3, change=align)
    x = torch.randn((total, width), generator=torch.Generator().manual_seed(3)).to(dtype)
    pairs = [(0, 100), (7, 200), (8, 255), (15, 256), (1, 330), (64, 390), (63, 401), (0, 419)]  # the last four are decoded
    for early, late in pairs:
        x[late] = x[early]
    probabilities = []
    expected = plain.latent_attention(x.double(), w, raw, "a.", 1e-5, kind == NEIGHBOURS, probabilities)
    heavy = max(float(p[late, early]) for p in probabilities for early, late in pairs[:1])
    assert heavy > 0.2 and all(max(float(p[late, early]) for p in probabilities) > 0.2 for early, late in pairs)
    session = Session([part.cache_need()], dtype, page_size=page, num_pages=-(-total // page) + 1, num_slots=2)
    for cuts in ([total], [330] + [1] * 90, [99, 2, 150, 69] + [1] * 50 + [2] * 25):
        close(dtype, _run_part(part, session, x, cuts), expected, f"cut as {cuts[:4]}...")


# the three forms of a step's runs through the state: a chain of chunks, chunks side by side, token by token
FORMS = (dict(chain_limit=10 ** 9), dict(chain_limit=0), dict(walk_limit=10 ** 9))


@pytest.mark.gpu
@pytest.mark.parametrize("spread", ["mild", "harsh"])
@pytest.mark.parametrize("heads,dim,vdim,rank,tau", [(4, 16, 8, 16, 16.0), (3, 40, 20, 5, 2.0), (2, 128, 64, 16, 1.0), (1, 256, 80, 32, 4.0),
                                                     (1, 3, 5, 1, 1.0), (2, 1, 300, 3, 8.0), (1, 20, 1100, 4, 3.0), (1, 500, 12, 8, 2.0), (2, 128, 256, 8, 16.0)])
def test_runs_in_chunks_as_token_by_token(heads, dim, vdim, rank, tau, spread):
    """Six requests (a run that ends inside a piece of a chunk, on a chunk's edge, one behind it, several chunks, a single
    token) from states that are not zero: the three forms and a plain loop agree on the normed and gated outputs and on the
    states they leave.  ``harsh``: decays down to e^-40 a token next to ones that keep everything, so that a piece of a chunk
    cannot be scored through factors."""
    from part_helpers import Session
    from kirai_b200.csrc import ops
    from kirai_b200.parts.base import StateNeed

    gen = torch.Generator().manual_seed(heads * 100 + dim)
    lens = [9, 64, 65, 200, 1, 33]
    T, keys, values = sum(lens), heads * dim, heads * vdim
    L = keys * vdim
    session = Session([StateNeed((L,), torch.float32)], torch.float32, page_size=4, num_pages=4, num_slots=8)
    batch = session.batch([(f"r{i}", n) for i, n in enumerate(lens)])
    rows = torch.randn((T, 2 * keys + 2 * values + rank), generator=gen)
    up, bias = torch.randn((rank, keys), generator=gen), torch.randn(keys, generator=gen)
    if spread == "harsh":
        up, bias = up * 12.0 * tau / rank ** 0.5, bias * 8.0 * tau
    norm = (1.0 + 0.3 * torch.randn(vdim, generator=gen)).repeat(heads)
    state0 = torch.randn((8, L), generator=gen)
    starts = batch.query_start.cpu().tolist()  # (the batch orders its requests itself)
    low = rows[:, 2 * keys + 2 * values :].double()
    log_a = (torch.nn.functional.logsigmoid(low @ up.double() + bias.double()) / tau).view(T, heads, dim)
    if spread == "harsh":
        assert float(log_a.min()) < -10.0 and float(log_a.max()) > -1e-3
    q, k = rows[:, :keys].double().view(T, heads, dim) * dim ** -0.5, rows[:, keys : 2 * keys].double().view(T, heads, dim)
    v, gate = rows[:, 2 * keys : 2 * keys + values].double().view(T, heads, vdim), rows[:, 2 * keys + values : 2 * keys + 2 * values].double()
    expected, states = torch.zeros((T, values), dtype=torch.float64), {}
    for r, (first, last) in enumerate(zip(starts, starts[1:])):
        slot = int(batch.slots[r])
        o, states[slot] = plain.linear_recurrence(q[first:last], k[first:last], v[first:last], log_a[first:last],
                                                  state0[slot].double().view(heads, dim, vdim))
        o = plain.unit_norm(o, norm[:vdim].double(), 1e-3)
        expected[first:last] = o.reshape(last - first, values) * plain.silu(gate[first:last])
    for limits in FORMS:
        st = state0.clone().cuda()
        got = ops.channel_scan(rows.cuda(), up.cuda(), bias.cuda(), tau, dim ** -0.5, st, batch, heads, dim, vdim, norm.cuda(), 1e-3,
                               torch.float32, **limits).cpu()
        assert float((got.double() - expected).abs().max()) <= 1e-4 * max(1.0, float(expected.abs().max())), limits
        for slot in range(8):
            want = states.get(slot, state0[slot].double().view(heads, dim, vdim))
            assert float((st[slot].cpu().double().view(heads, dim, vdim) - want).abs().max()) <= 3e-5 * max(1.0, float(want.abs().max())), (limits, slot)
    # single tokens: every request's first row, from the same states (a state's rows in registers where they fit)
    single = Session([StateNeed((L,), torch.float32)], torch.float32, page_size=4, num_pages=8, num_slots=8).batch([(f"r{i}", 1) for i in range(6)])
    firsts = torch.tensor(starts[:-1])
    st = state0.clone().cuda()
    got = ops.channel_scan(rows[firsts].contiguous().cuda(), up.cuda(), bias.cuda(), tau, dim ** -0.5, st, single, heads, dim, vdim, norm.cuda(), 1e-3,
                           torch.float32).cpu()
    for r, first in enumerate(firsts.tolist()):
        slot = int(single.slots[r])
        one = slice(first, first + 1)
        o, S = plain.linear_recurrence(q[one], k[one], v[one], log_a[one], state0[slot].double().view(heads, dim, vdim))
        want = plain.unit_norm(o, norm[:vdim].double(), 1e-3).reshape(1, values) * plain.silu(gate[one])
        assert float((got[r].double() - want).abs().max()) <= 1e-4 * max(1.0, float(want.abs().max())), ("single", r)
        assert float((st[slot].cpu().double().view(heads, dim, vdim) - S).abs().max()) <= 3e-5 * max(1.0, float(S.abs().max())), ("single", slot)
    narrow = ops.channel_scan(rows.cuda(), up.cuda(), bias.cuda(), tau, dim ** -0.5, state0.clone().cuda(), batch, heads, dim, vdim, norm.cuda(),
                              1e-3, torch.bfloat16)
    assert narrow.dtype == torch.bfloat16
    close(torch.bfloat16, narrow.float().cpu(), expected, "bfloat16 rows out")


GLA_CASES = [(2, 24, 16, 8.0, 64), (3, 20, 12, 2.0, 100), (1, 1, 37, 16.0, 40), (1, 70, 6, 1.0, 48), (4, 8, 32, 3.0, 72)]  # heads, dim, vdim, tau, width


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", GLA_CASES, ids=lambda c: "x".join(map(str, c)))
def test_linear_attention_whole_in_portions_and_one_by_one(dtype, case):
    """The state carries from step to step and starts at zero in a slot that an earlier request left.  A state that is lost
    between steps, or decays without their root, is far outside the bound."""
    from part_helpers import Session

    *sizes, width = case
    part, raw = _mixer(gla(*sizes), width)
    w = _loaded(part, dtype, width)
    xs = _unequal_rows(width, 3, dtype)
    expected = {name: plain.gated_linear_attention(x.double(), w, raw, "a.", 1e-5) for name, x in xs.items()}
    x = xs["p"].double()
    lost = torch.cat([plain.gated_linear_attention(x[:35], w, raw, "a.", 1e-5), plain.gated_linear_attention(x[35:], w, raw, "a.", 1e-5)])
    assert float((lost - expected["p"]).abs().max()) > tolerance("bfloat16", expected["p"].numpy())
    other = plain.gated_linear_attention(x, w, {**raw, "tau": raw["tau"] * 1.5}, "a.", 1e-5)
    assert float((other - expected["p"]).abs().max()) > 20 * tolerance("float32", expected["p"].numpy())
    session = Session([part.cache_need()], dtype, page_size=4, num_pages=40, num_slots=2)
    for cuts in CUTS(70):
        close(dtype, _run_part(part, session, xs["p"], cuts), expected["p"], f"cut as {cuts[:4]}...")
    got = _run_together(part, session, xs, UNEQUAL)
    for name in xs:
        close(dtype, got[name], expected[name], f"request {name} in batches")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_linear_attention_over_a_long_prompt_and_long_decoding(dtype):
    """600 tokens; channels that keep for hundreds of tokens beside ones that forget at once.  The first token's key and value
    are large, and the last queries still read them."""
    from part_helpers import Session

    part, raw = _mixer(gla(2, 32, 24, 4.0), 48)

    def keep(tensors):
        b = tensors["a.a2.b"].float().view(2, 32)
        b[:, ::2] = 12.0
        tensors["a.a2.b"] = b.reshape(-1).to(torch.bfloat16)
        tensors["a.a2"] = (tensors["a.a2"].float().view(2, 32, -1) * torch.tensor([0.1, 1.0]).repeat(16)[None, :, None]).reshape(64, -1).to(torch.bfloat16)

    w = _loaded(part, dtype, 7, change=keep)
    x = torch.randn((600, 48), generator=torch.Generator().manual_seed(8)).to(dtype)
    x[0] *= 12.0
    expected = plain.gated_linear_attention(x.double(), w, raw, "a.", 1e-5)
    without = plain.gated_linear_attention(torch.cat([x[:1] * 0.0, x[1:]]).double(), w, raw, "a.", 1e-5)
    assert float((without - expected)[-40:].abs().max()) > tolerance("bfloat16", expected.numpy())
    session = Session([part.cache_need()], dtype, page_size=4, num_pages=150, num_slots=1)
    for cuts in ([600], [300, 1, 299], [64] * 9 + [24], [250] + [1] * 350):
        close(dtype, _run_part(part, session, x, cuts), expected, f"cut as {cuts[:3]}")


def _feed_forward(mlp, width):
    import kirai_b200  # noqa: F401
    from kirai_b200.config.damilix import DamilixConfig
    from kirai_b200.models.damilix import feed_forward_for_layer

    raw = {"architecture": "Damilix", "width": width, "vocab": 16, "norm": {"eps": 1e-4}, "token_side": {"dim": 4},
           "layers": [layer(gla(1, 2, 2, 1.0), mlp)]}
    cfg = DamilixConfig.from_dict(raw)
    return feed_forward_for_layer(cfg, cfg.layers[0], "a.")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,identity,top,extra,tokens", [(8, 2, 3, 1, 5), (8, 2, 3, 0, 700), (1, 0, 1, 1, 3), (40, 24, 6, 1, 100), (3, 5, 8, 0, 9)])
def test_router_choice_weights_and_the_columns_behind(dtype, experts, identity, top, extra, tokens):
    """Choices, weights and the sigmoid columns against the plain rule, for the kernels of few and many tokens and for logits
    that a product left; the choice differs from one without the correction, the weights from uncorrected scores."""
    from kirai_b200.csrc import ops

    E, width = experts + identity, 64
    g = torch.Generator().manual_seed(E)
    x = torch.randn((tokens, width), generator=g).to(dtype)
    matrix = (torch.randn((E + extra, width), generator=g) * 0.4).to(torch.bfloat16)
    correction = torch.randn(E, generator=g) * 0.2
    w = {"m.router": matrix[:E].double(), "m.correction": correction.double()}
    margins = []
    ids, weights = plain.router_choice(x.double(), w, moe(4, experts, top, 1.7, identity=identity), "m.", margins)
    sure = margins[0] > 1e-4
    assert int(sure.sum()) >= tokens * 0.9
    if top < E and tokens > 4:
        bare, _ = plain.router_choice(x.double(), {**w, "m.correction": 0.0 * w["m.correction"]}, moe(4, experts, top, 1.7, identity=identity), "m.")
        assert not torch.equal(bare.sort(-1).values, ids.sort(-1).values)
    rule = {"correction": correction.cuda(), "scale": 1.7, "extra": extra}
    logits = x.double() @ matrix.double().T
    results = [ops.router_gates(x.cuda(), matrix.float().cuda(), top, True, rule=rule), ops.router_choose_(logits.float().cuda(), top, True, rule=rule)]
    dense = torch.zeros((tokens, E), dtype=torch.float64).scatter_(1, ids, weights)
    for gates, got_ids, got_weights in results:
        assert gates.shape == (tokens, E + extra)
        assert torch.equal(got_ids.cpu().long()[sure], ids[sure])
        assert float((got_weights.cpu().double() - weights)[sure].abs().max()) < 2e-5
        assert float((gates[:, :E].cpu().double() - dense)[sure].abs().max()) < 2e-5
        if extra:
            assert float((gates[:, E].cpu().double() - torch.sigmoid(logits[:, E])).abs().max()) < 2e-5


MOE_CASES = [  # mlp, width: stacked shared branch; sizes that cannot be stacked; no shared branch; one expert a token; sorted by expert
    (moe(16, 8, 3, 1.7, identity=2, shared=24), 64), (moe(12, 5, 2, 0.8, identity=3, shared=21), 100), (moe(20, 4, 3, 1.4, shared=12), 72),
    (moe(32, 3, 1, 1.0), 48), (moe(8, 2, 2, 1.2, identity=1), 36), (moe(128, 6, 2, 2.0, identity=2, shared=256), 128),
    (moe(256, 4, 3, 0.9), 384), (moe(128, 3, 2, 1.1, identity=4, shared=36), 256)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp,width", MOE_CASES, ids=lambda c: str(c) if isinstance(c, int) else f"{c['expert']['ff']}x{c['router']['experts']}")
def test_experts_identity_experts_and_the_gated_shared_branch(dtype, mlp, width):
    """The sum alone and added through a norm into the stream, for few tokens and for enough that rows are sorted by expert.
    An identity expert left out, a shared branch without its gate or weights without their factor lie far outside the bound."""
    from part_helpers import DEV
    from kirai_b200.parts import RMSNorm
    from part_helpers import load_part

    part = _feed_forward(mlp, width)
    w = _loaded(part, dtype, width)
    norm = RMSNorm("n", width, 1e-4)
    wn = load_part(norm, dtype, seed=width)["n"].double()
    tokens = 700
    stream = torch.randn((tokens, width), generator=torch.Generator().manual_seed(width)) * 1.5
    x = stream.to(dtype)
    margins = []
    expected = plain.routed_ffn(x.double(), w, mlp, "a.", margins)
    sure = (margins[0] > (1e-4 if dtype == torch.float32 else 5e-3))
    assert int(sure.sum()) > 0.8 * tokens
    bound = tolerance(dtype, expected[sure].numpy())
    if mlp["router"].get("identity"):
        other = plain.routed_ffn(x.double(), w, {**mlp, "router": {**mlp["router"], "experts": mlp["router"]["experts"], "scale": mlp["router"]["scale"] * 1.3}}, "a.")
        assert float((other - expected)[sure].abs().max()) > 2 * bound
        assert bool((plain.router_choice(x.double(), w, mlp, "a.")[0] >= mlp["router"]["experts"]).any())
    if mlp.get("shared"):
        other = plain.routed_ffn(x.double(), {**w, "a.shared.sg": 0.0 * w["a.shared.sg"]}, mlp, "a.")
        assert float((other - expected)[sure].abs().max()) > 2 * bound
    for rows in (1, 7, 60, 300, tokens):
        keep = sure[:rows]
        got = part.forward(x[:rows].to(DEV), None).cpu()
        assert got.dtype == torch.float32
        if bool(keep.any()):
            assert float((got.double() - expected[:rows])[keep].abs().max()) <= bound, rows
        if not part.adds_normed(rows) or dtype == torch.float32 or norm.fused_spec() is None:
            continue
        resid = stream[:rows].to(DEV)
        copy = part.forward_add_normed(x[:rows].to(DEV), None, resid, norm.fused_spec())
        added = plain.unit_norm(expected[:rows], wn, 1e-4)
        if bool(keep.any()):
            assert float((resid.cpu().double() - stream[:rows].double() - added)[keep].abs().max()) <= tolerance(dtype, added.numpy()), rows
        assert torch.equal(copy, resid.to(torch.bfloat16))


def test_experts_refuse_options_that_do_not_fit():
    import kirai_b200  # noqa: F401
    from kirai_b200.parts import GatedMLP, RoutedExperts

    shared = GatedMLP("s.", 16, 8)
    good = dict(activation="silu_gated", scoring="softmax_corrected", weight_scale=1.0)
    assert RoutedExperts("a.", 16, 8, 4, 2, **good, identity=2).routes == 6
    for bad in (dict(good, weight_scale=None), dict(good, activation="relu2"), dict(good, shared=shared), dict(good, shared_gate="sg"),
                dict(activation="silu_gated", identity=1), dict(activation="silu_gated", correction=True)):
        with pytest.raises(ValueError):
            RoutedExperts("a.", 16, 8, 4, 2, **bad)


# --------------------------------------------------------------------------- whole models (GPU)
def plain_reference(config, weights, tokens):
    """(logits of every token; the bound on each row's error in 32-bit and in bfloat16; which tokens chose their experts by more
    than rounding to bfloat16 can close).  A norm behind a state that a head has just begun to fill, or an attention that
    hangs between two keys, makes some rows sensitive whatever computes them: a row's bound follows what changing the weights'
    last bits does to it in the plain model, where that is more than the common bound."""
    margins = []
    logits = plain.forward(config, weights, tokens, margins=margins).numpy()
    gaps = torch.stack(margins)
    moved, shaken = np.zeros(len(tokens)), torch.zeros_like(gaps)
    for seed in range(3):
        g = torch.Generator().manual_seed(seed)
        other = {k: v.double() * (1.0 + torch.randn(v.shape, generator=g, dtype=torch.float64) * 2.0 ** -9) for k, v in weights.items()}
        margins = []
        moved = np.maximum(moved, np.abs(plain.forward(config, other, tokens, margins=margins).numpy() - logits).max(axis=1))
        shaken = torch.maximum(shaken, (torch.stack(margins) - gaps).abs())
    sure = (gaps > torch.clamp(3.0 * shaken, min=0.004)).all(dim=0)
    assert int(sure.sum()) >= 0.3 * len(tokens)
    bounds = {"bfloat16": np.maximum(tolerance("bfloat16", logits), 3.0 * moved),
              "float32": np.maximum(tolerance("float32", logits), moved * 2.0 ** -12)}
    return logits, bounds, sure.numpy()


def long_reference(tiny, tokens):
    """``plain_reference`` of a sequence, worked out once for both precisions."""
    known = tiny.setdefault("long", {})
    if tuple(tokens) not in known:
        known[tuple(tokens)] = plain_reference(tiny["config"], tiny["weights"], tokens)
    return known[tuple(tokens)]


def check(dtype, got, reference, rows, what):
    logits, bounds, sure = reference
    rows = np.asarray(list(rows))
    assert got.shape == (len(rows), logits.shape[1]), what
    assert np.isfinite(got).all(), what
    over = np.abs(got - logits[rows]).max(axis=1) / bounds[dtype][rows]
    if dtype == "bfloat16":
        over = over[sure[rows]]
    if over.size:
        assert over.max() <= 1.0, f"{what}: {over.max()} of the bound"


@pytest.fixture(scope="module", params=["A", "B", "C"])
def tiny(request, tmp_path_factory):
    raw, page, seed = TINY[request.param]
    folder = str(tmp_path_factory.mktemp(f"damilix{request.param}"))
    write_model(folder, raw, seed)
    config, weights = read_model_folder(folder)
    assert config == raw
    sequences = {rid: random_tokens(n, raw["vocab"], 300 + k)
                 for k, (rid, n) in enumerate([("a", 75), ("b", 40), ("c", 53), ("d", 9), ("e", 61), ("f", 34)])}
    reference = {rid: plain_reference(config, weights, toks) for rid, toks in sequences.items()}
    return dict(name=request.param, folder=folder, raw=raw, config=config, weights=weights, page=page,
                sequences=sequences, reference=reference)


@pytest.mark.gpu
def test_stream_after_every_layer(tiny):
    """In 32-bit the stream after each layer equals the plain one."""
    from kirai_b200.engine.batch import StepEntry
    from kirai_b200.engine.runner import ModelRunner
    from kirai_b200.parts.block import Block

    runner = ModelRunner.from_folder(tiny["folder"], dtype="float32", page_size=tiny["page"], max_tokens=128, num_slots=2)
    tokens = tiny["sequences"]["b"]
    _, streams = plain.forward(tiny["config"], tiny["weights"], tokens, keep_layers=True)
    kept, original = [], Block.forward

    def recording(self, resid, *args, **kwargs):
        resid, left = original(self, resid, *args, **kwargs)
        kept.append(resid.cpu().clone())
        return resid, left

    Block.forward = recording
    try:
        runner.step([StepEntry(runner.cache.open("b"), tokens, [0])])
    finally:
        Block.forward = original
    assert len(kept) == len(streams)
    for index, stream in enumerate(kept):
        assert float((stream - streams[index]).abs().max()) < 2e-4 * max(1.0, float(streams[index].abs().max())), f"after layer {index}"


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
    """A prompt of many chunks whole and beside a second request; the same prompt in portions; both against the plain model."""
    from replay_client import Replay

    toks = random_tokens(330, tiny["raw"]["vocab"], 77)
    other = tiny["sequences"]["d"]
    reference = long_reference(tiny, toks)
    rows = [0, 1, 15, 16, 63, 64, 65, 127, 128, 200, 255, 256, 257, 300, 328, 329]
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
    """Portions that end inside a page and inside a chunk's pieces."""
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
    """330 tokens one by one from the first."""
    from replay_client import Replay

    toks = random_tokens(330, tiny["raw"]["vocab"], 17)
    reference = long_reference(tiny, toks)
    replay = Replay(tiny["folder"], dtype, str(tmp_path / "out"), max_tokens=352, page_size=tiny["page"])
    for i, token in enumerate(toks):
        got = replay.step([("long", [token], [0])])
        check(dtype, got, reference, [i], f"decode at {i}")
    assert replay.close() == 0


def test_bounds_would_show_a_fault_in_each_mechanism(tiny):
    """What each of these faults costs a whole model's logits, against the bfloat16 bound of its tests."""
    tokens, weights = tiny["sequences"]["a"], tiny["weights"]
    true, bounds, sure = tiny["reference"]["a"]

    def with_patched(name, replacement):
        original = getattr(plain, name)
        setattr(plain, name, replacement(original))
        try:
            return plain.forward(tiny["config"], weights, tokens).numpy()
        finally:
            setattr(plain, name, original)

    def changed(suffix, factor):
        return plain.forward(tiny["config"], {k: v * factor if k.endswith(suffix) else v for k, v in weights.items()}, tokens).numpy()

    faults = {
        "no sink": with_patched("sink_softmax", lambda f: lambda s, see, sink: f(s, see, sink - 60.0)),
        "no state": with_patched("linear_recurrence", lambda f: lambda q, k, v, g: f(q, k, v, g - 60.0)),
        "no decay": with_patched("log_decays", lambda f: lambda *a: 0.0 * f(*a)),
        "no input of the token's own": with_patched("token_input", lambda f: lambda *a: 0.0 * f(*a)),
        "no rotation": with_patched("rotate", lambda f: lambda x, p, r, n: x),
        "no correction": changed(".correction", 0.0),
    }
    if any("identity" in (entry["mlp"] or {}).get("router", {}) for entry in tiny["raw"]["layers"]):
        faults["identity experts give nothing"] = with_patched("router_choice", lambda f: lambda x, w, mlp, p, m=None: (
            lambda ids, weight: (ids, weight * (ids < mlp["router"]["experts"])))(*f(x, w, mlp, p, m)))
    if any("shared" in (entry["mlp"] or {}) for entry in tiny["raw"]["layers"]):
        faults["a shared branch without its gate"] = changed(".shared.sg", 0.0)
    costs = {name: float((np.abs(other - true).max(axis=1) / bounds["bfloat16"])[sure].max()) for name, other in faults.items()}
    assert min(costs.values()) > 1.0, costs


def _sure_tokens(config, weights, prompt, generated):
    """How many of the generated tokens, from the first on, are chosen by a margin that rounding to bfloat16 cannot close."""
    logits, bounds, experts = plain_reference(config, weights, list(prompt) + list(generated))
    top2 = torch.topk(torch.from_numpy(logits)[len(prompt) - 1 : -1], 2, dim=-1).values
    clear = (top2[:, 0] - top2[:, 1]).numpy() > bounds["bfloat16"][len(prompt) - 1 : -1]
    sure = (clear & experts[len(prompt) - 1 : -1]).tolist()
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
    assert compared >= (40 if dtype == "float32" else 1)
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
