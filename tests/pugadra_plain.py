"""The Pugadra decoder stated plainly from its equations: float64, one function per mechanism, whole
sequences with explicit masks, nothing of the package imported.

``forward(config, weights, tokens)`` gives the logits of every position of one sequence and the
residual stream after every layer; the engine's tests compare against it.

A norm in front of and behind every sublayer, a residual multiplier; windowed grouped-query attention
with biases, a short convolution over time on the projected queries, keys and values, neighbouring
dimensions rotated in pairs, one in the softmax's denominator, a gate per element on its output; layers
that use an earlier layer's keys and values; gated feed-forwards with clamped branches, dense or routed
with a shared expert; a second embedding per token and layer; the embedding table as output matrix.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64
#: the design's fixed number: the factor inside the sigmoid of a feed-forward's gate
GATE_SLOPE = 1.702


def root_mean_square(x, eps):
    return torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def norm_around_one(x, weight, eps):
    """The stored weight is what is added to one."""
    return x / root_mean_square(x, eps) * (1.0 + weight)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z.pow(3))))


def causal_convolution(u, taps):
    """u [T, channels], taps [channels, n]: the last tap weighs the token itself, the ones before it the
    tokens before; nothing lies ahead of the sequence."""
    length, n = u.shape[0], taps.shape[1]
    padded = torch.cat([u.new_zeros(n - 1, u.shape[1]), u])
    return sum(padded[j:j + length] * taps[:, j] for j in range(n))


def rotate_neighbours(x, positions, rot):
    """x [T, heads, size]: of the first ``dims`` dimensions 2i and 2i + 1 are a pair, the rest stay."""
    if rot is None:
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    table = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=x.dtype)
    angle = torch.as_tensor(positions, dtype=x.dtype)[:, None, None] * table
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * torch.cos(angle) - v * torch.sin(angle)
    out[..., 1:dims:2] = v * torch.cos(angle) + u * torch.sin(angle)
    return out


def visible(length, size):
    """[T, T]: whether query i sees key j."""
    i, j = torch.arange(length)[:, None], torch.arange(length)[None, :]
    mask = j <= i
    return mask if size is None else mask & (i - j < size)


def softmax_plus_one(scores, mask):
    """exp(s) over one plus their sum."""
    scores = torch.where(mask, scores, torch.full_like(scores, -math.inf))
    top = torch.clamp(scores.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(scores - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def projected(h, w, name):
    """A projection with its bias, then its convolution."""
    return causal_convolution(h @ w[name].T + w[name + ".b"], w[name + ".conv"])


def attention(h, w, m, shared=None):
    """Returns the mixer's output and the (rotated) keys and values it used; ``shared``: another layer's."""
    length = h.shape[0]
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    positions = list(range(length))
    q = rotate_neighbours(projected(h, w, "q").view(length, heads, dim), positions, m.get("rot"))
    if shared is None:
        k = rotate_neighbours(projected(h, w, "k").view(length, groups, dim), positions, m.get("rot"))
        v = projected(h, w, "v").view(length, groups, vdim)
        shared = (k, v)
    k, v = (t.repeat_interleave(heads // groups, dim=1) for t in shared)
    scores = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"])
    p = softmax_plus_one(scores, visible(length, (m.get("mask") or {}).get("size")))
    mixed = torch.einsum("hij,jhv->ihv", p, v).reshape(length, heads * vdim)
    return (mixed * torch.sigmoid(h @ w["g"].T)) @ w["o"].T, shared


def clamped_gate(h, w, limit):
    """A feed-forward whose branches are clamped: the gate from above, the other one on both sides."""
    g = torch.clamp(h @ w["gate"].T, max=limit)
    u = torch.clamp(h @ w["up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(GATE_SLOPE * g) * (u + 1.0)) @ w["down"].T


def routed_feed_forward(h, w, mlp, margins=None):
    logits = h @ w["router"].T + w["router.b"]
    top, limit = int(mlp["router"]["top"]), float(mlp["expert"]["limit"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = torch.sort(logits[t], descending=True).indices.tolist()
        chosen, rest = order[:top], order[top:]
        if margins is not None:
            margins.append(float(logits[t, chosen[-1]] - logits[t, rest[0]]) if rest else math.inf)
        weights = torch.softmax(logits[t, chosen], dim=0)
        for e, share in zip(chosen, weights):
            out[t] += share * clamped_gate(h[t], _sub(w, f"e{e}."), limit)
    if mlp.get("shared") is not None:
        out = out + clamped_gate(h, _sub(w, "shared."), float(mlp["shared"]["limit"]))
    return out


def token_input(x, rows, w, eps):
    """What a layer adds for its tokens' rows of the second table, before the residual multiplier."""
    y = (gelu_tanh(x @ w["gate"].T) * rows) @ w["proj"].T
    return y / root_mean_square(y, eps) * w["norm"]


def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens, dtype=F64, margins=None):
    """Logits ``[T, vocab]`` and the residual stream after every layer ``[layers, T, width]``."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, m = float(config["norm"]["eps"]), float(config["residual_mult"])
    ids = torch.tensor(tokens)
    x = w["embed"][ids]
    after, kept = [], {}
    for index, layer in enumerate(config["layers"]):
        lw = _sub(w, f"l{index}.")
        y, kept[index] = attention(norm_around_one(x, lw["norm1"], eps), _sub(lw, "mix."), layer["mixer"],
                                   kept.get(layer["mixer"].get("kv_from")))
        x = x + m * norm_around_one(y, lw["norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h, mw = norm_around_one(x, lw["norm2"], eps), _sub(lw, "mlp.")
            y = clamped_gate(h, mw, float(mlp["limit"])) if mlp["kind"] == "dense" else \
                routed_feed_forward(h, mw, mlp, margins)
            x = x + m * norm_around_one(y, lw["norm2b"], eps)
        if config.get("token_side") is not None:
            size = int(config["token_side"]["dim"])
            x = x + m * token_input(x, w["side.embed"][ids, index * size:(index + 1) * size], _sub(lw, "side."), eps)
        after.append(x)
    return norm_around_one(x, w["final.norm"], eps) @ w["embed"].T, torch.stack(after)


# ---------------------------------------------------------------------------
def tensor_shapes(config):
    width, count = config["width"], len(config["layers"])
    shapes = {"embed": (config["vocab"], width), "final.norm": (width,)}
    side = config.get("token_side")
    if side is not None:
        shapes["side.embed"] = (config["vocab"], count * side["dim"])
    for index, layer in enumerate(config["layers"]):
        p, m, mlp = f"l{index}.", layer["mixer"], layer.get("mlp")
        heads, groups, dim, vdim, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp is not None else ()):
            shapes[p + name] = (width,)
        rows = {"q": heads * dim}
        if m.get("kv_from") is None:
            rows.update(k=groups * dim, v=groups * vdim)
        for name, size in rows.items():
            shapes.update({p + f"mix.{name}": (size, width), p + f"mix.{name}.b": (size,),
                           p + f"mix.{name}.conv": (size, taps)})
        shapes[p + "mix.g"] = (heads * vdim, width)
        shapes[p + "mix.o"] = (width, heads * vdim)
        if side is not None:
            shapes.update({p + "side.gate": (side["dim"], width), p + "side.proj": (width, side["dim"]),
                           p + "side.norm": (width,)})
        if mlp is None:
            continue
        parts = {"": mlp["ff"]} if mlp["kind"] == "dense" else \
            {f"e{e}.": mlp["expert"]["ff"] for e in range(mlp["router"]["experts"])}
        if mlp["kind"] == "moe":
            shapes[p + "mlp.router"] = (mlp["router"]["experts"], width)
            shapes[p + "mlp.router.b"] = (mlp["router"]["experts"],)
            if mlp.get("shared") is not None:
                parts["shared."] = mlp["shared"]["ff"]
        for part, ff in parts.items():
            shapes.update({p + f"mlp.{part}gate": (ff, width), p + f"mlp.{part}up": (ff, width),
                           p + f"mlp.{part}down": (width, ff)})
    return shapes


def random_model(config, seed):
    """Random bfloat16 weights that keep activations of order one: matrices N(0, 1/in), biases of half,
    norm weights around zero (the token input's around one), convolutions whose every tap counts."""
    generator = torch.Generator().manual_seed(seed)
    weights = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".")[-1]
        t = torch.randn(shape, generator=generator)
        if name.endswith("side.norm"):
            t = 1.0 + 0.1 * t
        elif "norm" in leaf:
            t = 0.2 * t
        elif leaf == "b":
            t = 0.5 * t
        elif leaf == "conv":
            t = t * shape[-1] ** -0.5
        elif leaf == "router":
            t = 2.0 * t * shape[-1] ** -0.5
        elif leaf != "embed":
            t = t * shape[-1] ** -0.5
        weights[name] = t.to(torch.bfloat16)
    return weights
