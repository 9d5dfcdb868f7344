"""The Sorizen decoder stated plainly from its equations: float64, one function per mechanism, whole
sequences with explicit masks, nothing of the package imported.

``forward(config, weights, tokens)`` gives the logits of every position of one sequence and the
sum of the residual streams after every run of a layer; the engine's tests compare against it.

Scaled token embedding; several residual streams that every sublayer reads through one vector and
writes through another while a matrix mixes them; layer norms with bias; latent attention with a
sliding window, either with a sink in the softmax's denominator or with a gate per head on its
output, keys rotated at stretched frequencies; dense feed-forwards with the exact GELU or routed
ones whose experts are chosen inside the groups with the best pairs of scores; layers that run
with another layer's tensors; the sum of the streams, final norm, an output matrix of its own.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64
#: what is added to the sum that the chosen experts' scores are divided by
SCORE_SUM_EPS = 1e-20


def rms_norm(x, weight, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * weight


def layer_norm(x, weight, bias, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt(centred.pow(2).mean(-1, keepdim=True) + eps) * weight + bias


def silu(z):
    return z * torch.sigmoid(z)


def gelu_exact(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def rotation_table(rot):
    """The frequency of every pair and the factor on both cosine and sine."""
    dims, base = int(rot["dims"]), float(rot["base"])
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if scaling is None:
        return plain, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def place(turns):
        """The (fractional) pair that makes that many turns over the original length."""
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(place(float(scaling["fast"]))), 0)
    high = min(math.ceil(place(float(scaling["slow"]))), dims - 1)
    table = []
    for i, f in enumerate(plain):
        ramp = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
        table.append(f / factor * ramp + f * (1.0 - ramp))
    return table, 0.1 * math.log(factor) + 1.0


def rotate_neighbours(x, positions, rot):
    """x [T, heads, dims]: dimensions 2i and 2i + 1 are a pair."""
    table, amplitude = rotation_table(rot)
    angle = torch.as_tensor(positions, dtype=x.dtype)[:, None, None] * torch.tensor(table, dtype=x.dtype)
    cos, sin = amplitude * torch.cos(angle), amplitude * torch.sin(angle)
    u, v = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., 0::2] = u * cos - v * sin
    out[..., 1::2] = v * cos + u * sin
    return out


def visible(length, size):
    """[T, T]: whether query i sees key j."""
    i, j = torch.arange(length)[:, None], torch.arange(length)[None, :]
    mask = j <= i
    return mask if size is None else mask & (i - j < size)


def attention_weights(scores, mask, sink=None):
    """scores [H, T, T]; ``sink`` [H] joins every denominator once, as a score with no value."""
    scores = torch.where(mask, scores, torch.full_like(scores, -math.inf))
    top = scores.max(dim=-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(scores - top)
    total = e.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink[:, None, None] - top)
    return e / total


def latent_attention(h, w, m, eps):
    """Both mixers: the one with a stored ``sink``, the other with an output gate ``g``."""
    length = h.shape[0]
    heads, dim, rot_dim, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = list(range(length))
    q = (h @ w["q"].T).view(length, heads, dim + rot_dim)
    q_plain, q_rot = q[..., :dim], rotate_neighbours(q[..., dim:], positions, m["rot"])
    down = h @ w["dkv"].T
    latent = rms_norm(down[:, :rank], w["dkv.norm"], eps)
    part = rotate_neighbours(down[:, None, rank:], positions, m["rot"])[:, 0]
    k = (latent @ w["uk"].T).view(length, heads, dim)
    v = (latent @ w["uv"].T).view(length, heads, vdim)
    scores = torch.einsum("ihd,jhd->hij", q_plain, k) + torch.einsum("ihr,jr->hij", q_rot, part)
    mask = visible(length, (m.get("mask") or {}).get("size"))
    p = attention_weights(scores * float(m["scale"]), mask, w.get("sink"))
    mixed = torch.einsum("hij,jhv->ihv", p, v)
    if "g" in w:
        mixed = mixed * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return mixed.reshape(length, -1) @ w["o"].T


def dense_feed_forward(h, w):
    return gelu_exact(h @ w["up"].T) @ w["down"].T


def expert(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def group_scores(scores, count):
    """A group of neighbours counts as much as its two best members together."""
    per = scores.shape[0] // count
    return torch.sort(scores.view(count, per), dim=1, descending=True).values[:, :2].sum(dim=1)


def route(scores, top, groups=None):
    """The chosen experts of one token, best first."""
    allowed = torch.ones_like(scores, dtype=torch.bool)
    if groups is not None:
        count, keep = int(groups["count"]), int(groups["keep"])
        kept = torch.topk(group_scores(scores, count), keep).indices
        allowed = torch.zeros(count, scores.shape[0] // count, dtype=torch.bool)
        allowed[kept] = True
        allowed = allowed.reshape(-1)
    return torch.topk(torch.where(allowed, scores, torch.full_like(scores, -math.inf)), top).indices.tolist()


def route_margin(scores, chosen, groups=None):
    """How far the choice lies from another one: of groups, and of experts inside the open groups."""
    margin = math.inf
    allowed = torch.ones_like(scores, dtype=torch.bool)
    if groups is not None:
        count, keep = int(groups["count"]), int(groups["keep"])
        ordered = torch.sort(group_scores(scores, count), descending=True)
        if keep < count:
            margin = float(ordered.values[keep - 1] - ordered.values[keep])
        allowed = torch.zeros(count, scores.shape[0] // count, dtype=torch.bool)
        allowed[ordered.indices[:keep]] = True
        allowed = allowed.reshape(-1)
    rest = [float(scores[e]) for e in range(scores.shape[0]) if allowed[e] and e not in chosen]
    return min(margin, min(float(scores[e]) for e in chosen) - max(rest)) if rest else margin


def routed_feed_forward(h, w, mlp, margins=None):
    router = mlp["router"]
    scores = torch.sigmoid(h @ w["router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = route(scores[t], int(router["top"]), router.get("groups"))
        if margins is not None:
            margins.append(route_margin(scores[t], chosen, router.get("groups")))
        total = scores[t, chosen].sum() + SCORE_SUM_EPS
        for e in chosen:
            out[t] += float(router["scale"]) * scores[t, e] / total * expert(h[t], _sub(w, f"e{e}."))
    return out


def hyper_connection(streams, w, sublayer):
    """streams [S, T, width]; ``w``: what the sublayer reads (``in``), writes (``out``) and how the
    streams mix (``mix``, from the first index to the second)."""
    u = torch.einsum("s,stw->tw", w["in"], streams)
    y = sublayer(u)
    return torch.einsum("sr,stw->rtw", w["mix"], streams) + w["out"][:, None, None] * y


def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def owner(config, index):
    """The layer whose tensors layer ``index`` runs with."""
    while config["layers"][index].get("weights_of") is not None:
        index = config["layers"][index]["weights_of"]
    return index


def forward(config, weights, tokens, dtype=F64, margins=None):
    """Logits ``[T, vocab]`` and the sum of the streams after every layer ``[layers, T, width]``."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens)] * float(config["embedding"]["scale"])
    streams = torch.stack([x] * int(config["streams"]))
    after = []
    for index, layer in enumerate(config["layers"]):
        lw = _sub(w, f"l{owner(config, index)}.")
        mix = _sub(lw, "mix.")

        def mixer(u):
            return latent_attention(layer_norm(u, lw["norm1"], lw["norm1.b"], eps), mix, layer["mixer"], eps)

        streams = hyper_connection(streams, _sub(lw, "hc1."), mixer)
        if layer.get("mlp") is not None:
            mlp = _sub(lw, "mlp.")

            def feed_forward(u):
                h = layer_norm(u, lw["norm2"], lw["norm2.b"], eps)
                if layer["mlp"]["kind"] == "dense":
                    return dense_feed_forward(h, mlp)
                return routed_feed_forward(h, mlp, layer["mlp"], margins)

            streams = hyper_connection(streams, _sub(lw, "hc2."), feed_forward)
        after.append(streams.sum(0))
    x = layer_norm(streams.sum(0), w["final.norm"], w["final.norm.b"], eps)
    return x @ w["head"].T, torch.stack(after)


# ---------------------------------------------------------------------------
def tensor_shapes(config):
    width, streams = config["width"], config["streams"]
    shapes = {"embed": (config["vocab"], width), "head": (config["vocab"], width), "final.norm": (width,),
              "final.norm.b": (width,)}
    for index, layer in enumerate(config["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m, mlp = f"l{index}.", layer["mixer"], layer.get("mlp")
        heads, rot_dim, rank = m["heads"], m["rot_dim"], m["kv_rank"]
        for q in (1, 2) if mlp is not None else (1,):
            shapes.update({p + f"norm{q}": (width,), p + f"norm{q}.b": (width,), p + f"hc{q}.in": (streams,),
                           p + f"hc{q}.out": (streams,), p + f"hc{q}.mix": (streams, streams)})
        shapes.update({
            p + "mix.q": (heads * (m["dim"] + rot_dim), width), p + "mix.dkv": (rank + rot_dim, width),
            p + "mix.dkv.norm": (rank,), p + "mix.uk": (heads * m["dim"], rank), p + "mix.uv": (heads * m["vdim"], rank),
            p + "mix.o": (width, heads * m["vdim"])})
        if layer["type"] == "latent_attention":
            shapes[p + "mix.sink"] = (heads,)
        else:
            shapes[p + "mix.g"] = (heads, width)
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            shapes.update({p + "mlp.up": (mlp["ff"], width), p + "mlp.down": (width, mlp["ff"])})
            continue
        ff, experts = mlp["expert"]["ff"], mlp["router"]["experts"]
        shapes[p + "mlp.router"] = (experts, width)
        for e in range(experts):
            shapes.update({p + f"mlp.e{e}.gate": (ff, width), p + f"mlp.e{e}.up": (ff, width),
                           p + f"mlp.e{e}.down": (width, ff)})
    return shapes


def random_model(config, seed):
    """Random bfloat16 weights that keep activations of order one: matrices N(0, 1/in), norm weights
    around one with biases of a tenth, stream mixes near the identity with every entry its own."""
    generator = torch.Generator().manual_seed(seed)
    streams = int(config["streams"])
    weights = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".")[-1]
        t = torch.randn(shape, generator=generator)
        if leaf == "b":
            t = 0.1 * t
        elif leaf in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.1 * t
        elif leaf == "sink":
            t = 0.5 * t
        elif leaf == "in":
            t = (1.0 + 0.3 * t) / streams
        elif leaf == "out":
            t = 1.0 + 0.3 * t
        elif leaf == "mix" and len(shape) == 2 and ".hc" in name:
            t = torch.eye(streams) + 0.15 * t
        elif leaf == "router":
            t = 2.0 * t * shape[-1] ** -0.5
        elif name != "embed":
            t = t * shape[-1] ** -0.5
        weights[name] = t.to(torch.bfloat16)
    return weights
