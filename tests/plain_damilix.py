"""A plain, slow implementation of the Damilix decoder: whole sequences, no cache, one function per mechanism,
64-bit arithmetic on the CPU.  It shares no code with the framework; model folders are read with the plain reader
of ``plain_qwen3``.

Notation: T tokens, E the model width, x the residual stream [T, E], which every sub-layer reads as it is.
"""
import math

import torch

F = torch.float64


def unit_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def pair_frequencies(rot):
    """One frequency per pair of columns: f_i = base^(-2i/dims); with ``scaling`` the frequencies from index ``lo`` to
    ``hi`` slide from f_i to f_i / factor.  Returns (frequencies, the factor on cosine and sine)."""
    dims, base = rot["dims"], rot["base"]
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(freq, dtype=F), 1.0

    def index_of(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(sc["fast"])), 0)
    hi = min(math.ceil(index_of(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return torch.tensor(out, dtype=F), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot, neighbours):
    """x [T, heads, dims] with its column pairs rotated by position * f_i: columns 2i and 2i + 1 (``neighbours``), or i and
    i + dims / 2."""
    dims = rot["dims"]
    freq, amplitude = pair_frequencies(rot)
    # the angle is a 32-bit product of a 32-bit position and a 32-bit frequency in the design
    angle = (positions.to(torch.float32)[:, None] * freq.to(torch.float32)[None, :]).to(F)
    cos, sin = angle.cos()[:, None, :] * amplitude, angle.sin()[:, None, :] * amplitude
    first, second = (slice(0, dims, 2), slice(1, dims, 2)) if neighbours else (slice(0, dims // 2), slice(dims // 2, dims))
    u, v = x[..., first], x[..., second]
    y = torch.empty_like(x)
    y[..., first] = u * cos - v * sin
    y[..., second] = v * cos + u * sin
    return y


def sink_softmax(scores, visible, sink):
    """Softmax of every row over its visible columns, with exp(sink) added to the denominator."""
    scores = scores.masked_fill(~visible, float("-inf"))
    peak = torch.clamp(scores.max(-1, keepdim=True).values, min=sink)
    e = torch.exp(scores - peak)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - peak))


def latent_attention(x, w, m, prefix, eps, neighbours, probabilities=None):
    """Queries straight from x; keys and values of all heads from one normed latent a token, plus one rotated key part
    that the heads share; causal; a learned sink per head in the softmax's denominator; head h's output times
    sigmoid(W_g x)_h."""
    T = x.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = torch.arange(T)
    q = (x @ w[prefix + "q"].T).view(T, H, d + r)
    q_rot = rotate(q[..., d:], positions, m["rot"], neighbours)
    down = x @ w[prefix + "dkv"].T
    latent = unit_norm(down[:, :rank], w[prefix + "dkv.norm"], eps)
    shared = rotate(down[:, rank:].reshape(T, 1, r), positions, m["rot"], neighbours)[:, 0]
    keys = (latent @ w[prefix + "uk"].T).view(T, H, d)
    values = (latent @ w[prefix + "uv"].T).view(T, H, dv)
    gate = torch.sigmoid(x @ w[prefix + "g"].T)
    visible = positions[None, :] <= positions[:, None]
    heads = []
    for h in range(H):
        p = sink_softmax((q[:, h, :d] @ keys[:, h].T + q_rot[:, h] @ shared.T) * m["scale"], visible, w[prefix + "sink"][h])
        if probabilities is not None:
            probabilities.append(p)
        heads.append((p @ values[:, h]) * gate[:, h : h + 1])
    return torch.cat(heads, dim=1) @ w[prefix + "o"].T


def log_decays(x, w, m, prefix):
    """log alpha [T, heads, dim]: the logarithm of sigmoid(W_a2 (W_a1 x) + b) to the power 1 / tau."""
    z = (x @ w[prefix + "a1"].T) @ w[prefix + "a2"].T + w[prefix + "a2.b"]
    return torch.nn.functional.logsigmoid(z).view(x.shape[0], m["heads"], m["dim"]) / m["tau"]


def linear_recurrence(q, k, v, log_alpha, state=None):
    """S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t, per head; q, k, log_alpha [T, H, d], v [T, H, dv].  Returns (o, S)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F) if state is None else state.clone()
    out = []
    for t in range(T):
        S = torch.exp(log_alpha[t])[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def gated_linear_attention(x, w, m, prefix, eps):
    T, H, d, dv = x.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (x @ w[prefix + "q"].T).view(T, H, d) * d ** -0.5
    k = (x @ w[prefix + "k"].T).view(T, H, d)
    v = (x @ w[prefix + "v"].T).view(T, H, dv)
    o, _ = linear_recurrence(q, k, v, log_decays(x, w, m, prefix))
    o = unit_norm(o, w[prefix + "norm"], eps).reshape(T, H * dv)
    return (o * silu(x @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def gated_ffn(x, w, prefix):
    return (silu(x @ w[prefix + "gate"].T) * (x @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def router_choice(x, w, mlp, prefix, margins=None):
    """(chosen experts [T, top], their weights [T, top]): softmax over every expert, the identity ones included; the
    choice by score + correction, the weights the chosen scores divided by their sum, times a constant.  ``margins``
    collects, per token, the gap that decided the choice."""
    router = mlp["router"]
    top, E = router["top"], router["experts"] + router.get("identity", 0)
    score = torch.softmax(x @ w[prefix + "router"].T, dim=-1)
    ordered = (score + w[prefix + "correction"]).sort(dim=-1, descending=True)
    ids = ordered.indices[:, :top]
    if margins is not None:
        margins.append(ordered.values[:, top - 1] - ordered.values[:, top] if top < E else torch.full((x.shape[0],), float("inf"), dtype=F))
    chosen = score.gather(1, ids)
    return ids, chosen / (chosen.sum(-1, keepdim=True) + 1e-20) * router["scale"]


def routed_ffn(x, w, mlp, prefix, margins=None):
    ids, weights = router_choice(x, w, mlp, prefix, margins)
    out = torch.zeros_like(x)
    experts = mlp["router"]["experts"]
    for e in range(experts + mlp["router"].get("identity", 0)):
        rows, slot = (ids == e).nonzero(as_tuple=True)
        if rows.numel():
            y = gated_ffn(x[rows], w, f"{prefix}e{e}.") if e < experts else x[rows]
            out[rows] += weights[rows, slot][:, None] * y
    if mlp.get("shared"):
        out = out + torch.sigmoid(x @ w[prefix + "shared.sg"].T) * gated_ffn(x, w, prefix + "shared.")
    return out


def token_input(x, tokens, w, config, index, prefix, eps):
    """What layer ``index`` adds from its part of the tokens' own rows: unit_norm(W_proj (gelu_tanh(W_gate x) * e)) * weight."""
    dim = config["token_side"]["dim"]
    e = w["side.embed"][tokens][:, index * dim : (index + 1) * dim]
    g = gelu_tanh(x @ w[prefix + "gate"].T) * e
    return unit_norm(g @ w[prefix + "proj"].T, w[prefix + "norm"], eps)


def forward(config, weights, tokens, keep_layers=False, margins=None):
    """Logits [T, vocab] (float32) of a whole sequence; with ``keep_layers`` also the stream after every layer."""
    w = {name: t.to(F) for name, t in weights.items()}
    eps = config["norm"]["eps"]
    tokens = torch.as_tensor(list(tokens), dtype=torch.long)
    x = unit_norm(w["embed"][tokens], w["embed.norm"], eps)
    kept = []
    for index, layer in enumerate(config["layers"]):
        base, mlp = f"l{index}.", layer["mlp"]
        if layer["type"] == "gla":
            a = gated_linear_attention(x, w, layer["mixer"], base + "mix.", eps)
        else:
            a = latent_attention(x, w, layer["mixer"], base + "mix.", eps, layer["type"] == "latent_attention")
        x = x + unit_norm(a, w[base + "norm1"], eps)
        if mlp is not None:
            f = gated_ffn(x, w, base + "mlp.") if mlp["kind"] == "dense" else routed_ffn(x, w, mlp, base + "mlp.", margins)
            x = x + unit_norm(f, w[base + "norm2"], eps)
        x = x + token_input(x, tokens, w, config, index, base + "side.", eps)
        kept.append(x.to(torch.float32))
    logits = (unit_norm(x, w["final.norm"], eps) @ w["head"].T).to(torch.float32)
    return (logits, torch.stack(kept)) if keep_layers else logits
