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
# the attention kernels' tiles, stretched frequencies that reach the clamp on both sides, one key column.  C: sizes and
# counts of one (one head, one expert a token, tau 1, no identity expert, no shared branch), a latent narrower than a head.
CONFIG_A = {
    "architecture": "Damilix", "width": 64, "vocab": 200, "norm": {"eps": 1e-5}, "token_side": {"dim": 8},
    "layers": [
        layer(latent(NEIGHBOURS, 4, 16, 8, 24, 32, 1.1, base=300.0, scaling=(4.0, 32, 8.0, 1.0)), dense(96)),
        layer(gla(2, 24, 16, 8.0), moe(16, 8, 3, 1.7, identity=2, shared=24)),
        layer(latent(HALVES, 2, 24, 16, 8, 24, 0.9), None),
        layer(gla(4, 8, 32, 3.0), dense(40)),
        layer(latent(HALVES, 8, 8, 8, 16, 40, 1.4, base=500.0), moe(24, 6, 2, 2.2, identity=1, shared=40)),
    ],
}
CONFIG_B = {
    "architecture": "Damilix", "width": 100, "vocab": 131, "norm": {"eps": 1e-3}, "token_side": {"dim": 5},
    "layers": [
        layer(gla(3, 20, 12, 2.0), moe(12, 5, 2, 0.8, identity=3, shared=21)),
        layer(latent(HALVES, 5, 10, 6, 12, 18, 1.3, base=50.0), dense(33)),
        layer(latent(NEIGHBOURS, 3, 12, 10, 20, 22, 1.0, base=77.0, scaling=(2.0, 16, 4.0, 0.5)), moe(20, 4, 3, 1.4, shared=12)),
        layer(gla(1, 1, 37, 16.0), None),
    ],
}
CONFIG_C = {
    "architecture": "Damilix", "width": 48, "vocab": 90, "norm": {"eps": 1e-6}, "token_side": {"dim": 16},
    "layers": [layer(latent(NEIGHBOURS, 1, 32, 16, 40, 16, 0.8), moe(32, 3, 1, 1.0)), layer(gla(1, 70, 6, 1.0), moe(8, 2, 2, 1.2, identity=1))],
}
TINY = {"A": (CONFIG_A, 4, 21), "B": (CONFIG_B, 8, 22), "C": (CONFIG_C, 16, 23)}  # name -> (config, page size, seed)


def loud(tensors, raw):
    """Random weights made so that each mechanism shows: sinks of the size of large scores, biases and projections of the decays
    that spread them from forgetting at once to keeping for hundreds of tokens, routers whose scores lie far apart, corrections
    that change choices."""
    for name, t in list(tensors.items()):
        if name.endswith(".sink"):
            tensors[name] = (t.float() * 12.0 + 1.0).to(torch.bfloat16)
        elif name.endswith(".a2.b"):
            tensors[name] = (t.float() * 25.0 + 2.0).to(torch.bfloat16)
        elif name.endswith((".a1", ".a2", ".router")):
            tensors[name] = (t.float() * 3.0).to(torch.bfloat16)
        elif name.endswith((".mix.g", ".side.gate", ".shared.sg")):
            tensors[name] = (t.float() * 2.0).to(torch.bfloat16)
    return tensors


def write_model(folder, raw, seed, std=0.1):
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
