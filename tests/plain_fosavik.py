"""A plain, slow implementation of the Fosavik decoder: whole sequences, no cache, one function per mechanism,
64-bit arithmetic on the CPU.  It shares no code with the framework; model folders are read with the plain reader
of ``plain_qwen3``.

Notation: T tokens, E the model width, s the number of copies of the stream, n the normed rows [T, E] a sub-layer reads,
c the configuration as the dict that config.json holds, m one mixer's part of it, w a dict of tensors by name.
"""
import math

import torch

F = torch.float64


# ---- norms and activations --------------------------------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


# ---- several copies of the stream ---------------------------------------------------------------------------------
def streams_read(xs, w, prefix):
    """u [T, E], what a sub-layer's norm reads: the copies xs [s, T, E] weighted and added."""
    return (w[prefix + "in"][:, None, None] * xs).sum(0)


def streams_update(xs, y, w, prefix):
    """Every copy afresh from all the old ones and the sub-layer's output y: copy t takes mix[f, t] of copy f."""
    mix, out = w[prefix + "mix"], w[prefix + "out"]
    return torch.stack([(mix[:, t][:, None, None] * xs).sum(0) + out[t] * y for t in range(xs.shape[0])])


# ---- embedding ------------------------------------------------------------------------------------------------------
def embedded(w, tokens):
    return w["embed"][torch.tensor(tokens)] + w["pos"][: len(tokens)]


# ---- attention with two maps ---------------------------------------------------------------------------------------
def causal(T):
    i = torch.arange(T)
    return i[None, :] <= i[:, None]


def map_weight(w, m, prefix):
    """lambda: how much of the second map's output is taken away, one number for the layer."""
    return (torch.exp((w[prefix + "lq1"] * w[prefix + "lk1"]).sum()) - torch.exp((w[prefix + "lq2"] * w[prefix + "lk2"]).sum())
            + m["diff"])


def keys_and_values(n, w, m, prefix):
    """k [T, G, 2, d] and v [T, G, dv]."""
    T, G = n.shape[0], m["kv_heads"]
    return (n @ w[prefix + "k"].T).view(T, G, 2, m["dim"]), (n @ w[prefix + "v"].T).view(T, G, m["vdim"])


def two_map_attention(n, w, m, prefix, eps, kv):
    T = n.shape[0]
    H, G = m["heads"], m["kv_heads"]
    k, v = kv
    q = (n @ w[prefix + "q"].T).view(T, H, 2, m["dim"])
    lam, see = map_weight(w, m, prefix), causal(T)
    heads = []
    for h in range(H):
        g = h // (H // G)
        out = []
        for one in (0, 1):
            scores = (q[:, h, one] @ k[:, g, one].T) * m["scale"]
            out.append(torch.softmax(scores.masked_fill(~see, float("-inf")), dim=-1) @ v[:, g])
        heads.append(unit_rms(out[0] - lam * out[1], eps) * (1.0 - m["diff"]))
    return torch.cat(heads, dim=-1) @ w[prefix + "o"].T


# ---- the left side: attention over a window, a sink, values that are the keys --------------------------------------
def visible_keys(T, size, keep_first):
    """[T, T] bool: row i sees column j when j <= i and (i - j < size or j < keep_first)."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_with_sink(scores):
    """exp(s_j) / (1 + sum_j exp(s_j)) over the last axis; -inf where nothing is seen."""
    top = scores.max(-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(scores - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def sink_attention(n, w, m, prefix, eps):
    T = n.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    projected = (n @ w[prefix + "k"].T).view(T, G, d)
    q = rms_norm((n @ w[prefix + "q"].T).view(T, H, d), w[prefix + "q.norm"], eps)
    k = rms_norm(projected, w[prefix + "k.norm"], eps)
    gate = torch.sigmoid(n @ w[prefix + "g"].T)  # [T, H]
    see = visible_keys(T, m["mask"]["size"], m["mask"]["keep_first"])
    heads = []
    for h in range(H):
        g = h // (H // G)
        scores = ((q[:, h] @ k[:, g].T) * m["scale"]).masked_fill(~see, float("-inf"))
        heads.append((softmax_with_sink(scores) @ projected[:, g]) * gate[:, h : h + 1])
    return torch.cat(heads, dim=-1) @ w[prefix + "o"].T


# ---- the right side: a gated linear recurrence per channel ------------------------------------------------------------
def causal_convolution(x, taps_w, bias):
    """x [T, C]; taps_w [C, K], whose last column weighs the current token; zeros before the start."""
    T, C = x.shape
    K = taps_w.shape[1]
    padded = torch.cat([torch.zeros(K - 1, C, dtype=x.dtype), x], dim=0)
    out = bias.expand(T, C).clone()
    for j in range(K):
        out = out + padded[j : j + T] * taps_w[:, j]
    return out


def block_product(u, weight, bias):
    """u [T, W] in equal parts, each through a square matrix of its own: weight [parts, out, in]."""
    T, parts = u.shape[0], weight.shape[0]
    return (torch.einsum("tbi,boi->tbo", u.view(T, parts, -1), weight) + bias).reshape(T, -1)


def linear_recurrence(n, w, m, prefix):
    y = gelu_tanh(n @ w[prefix + "y"].T + w[prefix + "y.b"])
    u = causal_convolution(n @ w[prefix + "x"].T + w[prefix + "x.b"], w[prefix + "conv"], w[prefix + "conv.b"])
    r = torch.sigmoid(block_product(u, w[prefix + "ra"], w[prefix + "ra.b"]))
    i = torch.sigmoid(block_product(u, w[prefix + "ri"], w[prefix + "ri.b"]))
    log_a = -8.0 * r * softplus(w[prefix + "lam"])
    S = torch.zeros(u.shape[1], dtype=F)
    rows = []
    for t in range(u.shape[0]):
        S = torch.exp(log_a[t]) * S + torch.sqrt(-torch.expm1(2.0 * log_a[t])) * i[t] * u[t]
        rows.append(S)
    return (torch.stack(rows) * y) @ w[prefix + "o"].T


def parallel_mixer(n, w, m, prefix, eps):
    return (m["left_scale"] * sink_attention(n, w, m["left"], prefix + "left.", eps)
            + m["right_scale"] * linear_recurrence(n, w, m["right"], prefix + "right."))


# ---- the state-space mixer ----------------------------------------------------------------------------------------------
def state_space(n, w, m, prefix, eps):
    T = n.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    proj = n @ w[prefix + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner : 2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N :]
    xbc = silu(causal_convolution(xbc, w[prefix + "conv"], w[prefix + "conv.b"]))
    x = xbc[:, :inner].view(T, H, P)
    group = torch.arange(H) // (H // G)
    B = xbc[:, inner : inner + G * N].view(T, G, N)[:, group]
    C = xbc[:, inner + G * N :].view(T, G, N)[:, group]
    dt = softplus(dt + w[prefix + "dt_bias"])                       # [T, H]
    decay = torch.exp(-torch.exp(w[prefix + "A_log"]) * dt)         # [T, H]
    S = torch.zeros(H, N, P, dtype=F)
    rows = []
    for t in range(T):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        rows.append((torch.einsum("hnp,hn->hp", S, C[t]) + w[prefix + "D"][:, None] * x[t]).reshape(-1))
    y = torch.stack(rows) * silu(z)
    parts = m["norm_groups"]
    y = unit_rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * w[prefix + "norm"]
    return y @ w[prefix + "o"].T


# ---- the feed-forward ---------------------------------------------------------------------------------------------------
def clamped_ffn(n, w, mlp, prefix):
    limit = mlp["limit"]
    g = torch.clamp(n @ w[prefix + "gate"].T, max=limit)
    u = torch.clamp(n @ w[prefix + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[prefix + "down"].T


# ---- the model ----------------------------------------------------------------------------------------------------------
def forward(c, w, tokens, return_layers=False):
    """Logits [T, vocab] of a whole sequence (and the sum of the stream's copies after every layer)."""
    w = {name: (t.to(F) if t.is_floating_point() else t) for name, t in w.items()}
    eps = c["norm"]["eps"]
    x = embedded(w, tokens)
    xs = torch.stack([x] * c["streams"])
    kept, layers = {}, []
    for i, layer in enumerate(c["layers"]):
        base, m = f"l{i}.", layer["mixer"]
        n = rms_norm(streams_read(xs, w, base + "hc1."), w[base + "norm1"], eps)
        if layer["type"] == "attention":
            source = m.get("kv_from")
            kept[i] = kept[source] if source is not None else keys_and_values(n, w, m, base + "mix.")
            y = two_map_attention(n, w, m, base + "mix.", eps, kept[i])
        elif layer["type"] == "parallel":
            y = parallel_mixer(n, w, m, base + "mix.", eps)
        elif layer["type"] == "mamba2":
            y = state_space(n, w, m, base + "mix.", eps)
        else:
            raise ValueError(layer["type"])
        xs = streams_update(xs, y, w, base + "hc1.")
        if layer.get("mlp") is not None:
            n = rms_norm(streams_read(xs, w, base + "hc2."), w[base + "norm2"], eps)
            xs = streams_update(xs, clamped_ffn(n, w, layer["mlp"], base + "mlp."), w, base + "hc2.")
        layers.append(xs.sum(0))
    logits = rms_norm(xs.sum(0), w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(layers)) if return_layers else logits
