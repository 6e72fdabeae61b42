"""A plain, slow implementation of the Zugutar decoder in float64: one function per mechanism, whole
sequences at once, the recurrence token by token, no code shared with the package.

``weights`` maps the names of the design's own weight file (``embed``, ``l0.mix.left.q``,
``l1.mlp.e3.up``, ...) to tensors; ``config`` is the design's config.json as a dict.

Notation.  The stream starts as ``x = E[token]``; a layer has one norm, which both of its sublayers read,

    h = N(x),   x += mixer(h) + ff(h)      (without the second term where it has no feed-forward)

with N(x) = x / rms(x) * (1 + w); a range of layers may run several times in a row, ``E[token]`` being
added to x in front of every pass but the first; the logits are ``c E N(x)``.  Mixers: attention without
positions whose queries grow with the logarithm of their position, with a gate per output value; and two
mixers side by side, attention with normed, rotated queries and keys, a sink of score 0 and a gate per
head, beside Mamba-2's recurrence.  Feed-forward: a mixture of gated units whose weight multiplies what
an expert reads, beside a gated shared unit.
"""
import math

import torch

F = torch.float64


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return over_rms(x, eps) * weight.to(F)


def zero_centred_norm(x, w, eps):
    """The stored weight is the gain's distance from one."""
    return over_rms(x, eps) * (1.0 + w.to(F))


def product(h, w):
    return h @ w.to(F).T


def silu(z):
    return z * torch.sigmoid(z)


def rotate_half(x, rot):
    """x [T, heads, d]: of the first rot.dims values of a head, value i turns with value i + dims/2 by
    position * base^(-2i/dims)."""
    dims = int(rot["dims"])
    half = dims // 2
    frequency = float(rot["base"]) ** (-2.0 * torch.arange(half, dtype=F) / max(dims, 1))
    angle = torch.arange(x.shape[0], dtype=F)[:, None] * frequency[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def temperature(count, q_temp):
    """[T]: what the query at each position is multiplied by."""
    position = torch.arange(count, dtype=F)
    return 1.0 + float(q_temp["coef"]) * torch.log(torch.floor((position + 1.0) / float(q_temp["every"])) + 1.0)


def causal_softmax(scores, sink=False):
    """scores [H, T, T]; with a sink the denominator also holds exp(0)."""
    count = scores.shape[-1]
    scores = scores.masked_fill(torch.arange(count)[None, :] > torch.arange(count)[:, None], float("-inf"))
    top = scores.max(dim=-1, keepdim=True).values
    if sink:
        top = torch.clamp(top, min=0.0)
    weights = torch.exp(scores - top)
    return weights / (weights.sum(-1, keepdim=True) + (torch.exp(-top) if sink else 0.0))


def heads_of(h, w, name, count):
    rows = product(h, w[name])
    return rows.reshape(h.shape[0], count, rows.shape[1] // count)


def attend(q, k, v, scale, sink=False):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: [T, H, dv]; query head h reads key head h // (H / G)."""
    group = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(group, dim=1), v.repeat_interleave(group, dim=1)
    weights = causal_softmax(torch.einsum("ihd,jhd->hij", q, k) * float(scale), sink)
    return torch.einsum("hij,jhd->ihd", weights, v)


def plain_attention(h, w, p, m):
    """The mixer ``attention``: no rotation, scaled queries, a gate per output value."""
    q = heads_of(h, w, f"{p}.q", int(m["heads"]))
    k, v = heads_of(h, w, f"{p}.k", int(m["kv_heads"])), heads_of(h, w, f"{p}.v", int(m["kv_heads"]))
    q = q * temperature(h.shape[0], m["q_temp"])[:, None, None]
    out = attend(q, k, v, m["scale"]).reshape(h.shape[0], -1)
    return product(out * torch.sigmoid(product(h, w[f"{p}.g"])), w[f"{p}.o"])


def rotated_attention(h, w, p, m, eps):
    """The left mixer of ``parallel``: a norm per head, rotation, a sink, a gate per head."""
    q = rms_norm(heads_of(h, w, f"{p}.q", int(m["heads"])), w[f"{p}.q.norm"], eps)
    k = rms_norm(heads_of(h, w, f"{p}.k", int(m["kv_heads"])), w[f"{p}.k.norm"], eps)
    v = heads_of(h, w, f"{p}.v", int(m["kv_heads"]))
    out = attend(rotate_half(q, m["rot"]), rotate_half(k, m["rot"]), v, m["scale"], sink=True)
    out = out * torch.sigmoid(product(h, w[f"{p}.g"]))[:, :, None]
    return product(out.reshape(h.shape[0], -1), w[f"{p}.o"])


def causal_conv(x, weight, bias):
    """x [T, C]; the last tap is the current token's, zeros in front of the first."""
    taps = weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F), x])
    out = bias.to(F).expand_as(x).clone()
    for j in range(taps):
        out = out + weight[:, j].to(F) * padded[j:j + x.shape[0]]
    return out


def state_recurrence(x, b, c, dt, decay_rate, d):
    """x [T, H, P], b and c [T, H, N], dt [T, H]: per head ``S = exp(-rate dt) S + dt b x^T``,
    ``y = S^T c + d x``."""
    count, heads, size = x.shape
    state = torch.zeros(heads, b.shape[2], size, dtype=F)
    out = torch.zeros_like(x)
    for t in range(count):
        state = torch.exp(-decay_rate * dt[t])[:, None, None] * state + dt[t][:, None, None] * b[t][:, :, None] * x[t][:, None, :]
        out[t] = torch.einsum("hnp,hn->hp", state, c[t]) + d[:, None] * x[t]
    return out


def mamba2(h, w, p, m, eps):
    """The right mixer of ``parallel``."""
    heads, size, n, groups = (int(m[k]) for k in ("heads", "vdim", "state", "groups"))
    count, inner = h.shape[0], heads * size
    whole = product(h, w[f"{p}.in"])
    z, xbc, dt = whole[:, :inner], whole[:, inner:2 * inner + 2 * groups * n], whole[:, 2 * inner + 2 * groups * n:]
    xbc = silu(causal_conv(xbc, w[f"{p}.conv"], w[f"{p}.conv.b"]))
    x = xbc[:, :inner].reshape(count, heads, size)
    b = xbc[:, inner:inner + groups * n].reshape(count, groups, n).repeat_interleave(heads // groups, dim=1)
    c = xbc[:, inner + groups * n:].reshape(count, groups, n).repeat_interleave(heads // groups, dim=1)
    dt = torch.nn.functional.softplus(dt + w[f"{p}.dt_bias"].to(F), threshold=1e9)
    y = state_recurrence(x, b, c, dt, torch.exp(w[f"{p}.A_log"].to(F)), w[f"{p}.D"].to(F)).reshape(count, inner)
    y = (y * silu(z)).reshape(count, int(m["norm_groups"]), -1)
    return product(over_rms(y, eps).reshape(count, inner) * w[f"{p}.norm"].to(F), w[f"{p}.o"])


def side_by_side(h, w, p, m, eps):
    left = rms_norm(rotated_attention(h, w, f"{p}.left", m["left"], eps), w[f"{p}.left.out"], eps)
    right = rms_norm(mamba2(h, w, f"{p}.right", m["right"], eps), w[f"{p}.right.out"], eps)
    return 0.5 * (left + right)


def unit(h, w, p):
    return product(silu(product(h, w[f"{p}.gate"])) * product(h, w[f"{p}.up"]), w[f"{p}.down"])


def route(h, w, p, router):
    """(chosen [T, top], scores of the chosen [T, top], margin [T]): the margin is the gap between the last
    chosen logit and the best one left out."""
    top = int(router["top"])
    ranked = product(h, w[f"{p}.router"]).sort(dim=-1, descending=True)
    margin = ranked.values[:, top - 1] - ranked.values[:, top] if top < ranked.values.shape[1] else \
        torch.full((h.shape[0],), math.inf, dtype=F)
    return ranked.indices[:, :top], torch.sigmoid(ranked.values[:, :top]), margin


def mixture(h, w, p, mlp, margins=None):
    chosen, weights, margin = route(h, w, p, mlp["router"])
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        tokens, places = torch.where(chosen == e)
        if tokens.numel():
            # the weight multiplies what the expert reads
            out[tokens] += unit(weights[tokens, places][:, None] * h[tokens], w, f"{p}.e{e}")
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(product(h, w[f"{p}.shared.sg"])) * unit(h, w, f"{p}.shared")
    return out


def layer_runs(config):
    """(layer, adds the embedding output first) of every run, in order."""
    count, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(count)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    runs = [(i, False) for i in range(start)]
    for turn in range(times):
        runs += [(i, turn > 0 and i == start) for i in range(start, stop)]
    return runs + [(i, False) for i in range(stop, count)]


def forward(config, weights, tokens, return_layers=False, margins=None):
    """Logits [T, vocab] of one sequence; with `return_layers` also the stream after every layer run.  A list
    given as `margins` receives every router's margin [T]."""
    w = weights
    eps = float(config["norm"]["eps"])
    embedded = w["embed"].to(F)[torch.tensor(tokens)]
    x = embedded
    streams = []
    for index, again in layer_runs(config):
        layer, p = config["layers"][index], f"l{index}"
        if again:
            x = x + embedded
        h = zero_centred_norm(x, w[f"{p}.norm1"], eps)
        if layer["type"] == "attention":
            total = plain_attention(h, w, f"{p}.mix", layer["mixer"])
        elif layer["type"] == "parallel":
            total = side_by_side(h, w, f"{p}.mix", layer["mixer"], eps)
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp") is not None:
            total = total + mixture(h, w, f"{p}.mlp", layer["mlp"], margins)
        x = x + total
        streams.append(x.clone())
    logits = product(zero_centred_norm(x, w["final.norm"], eps), w["embed"]) * float(config["logit_scale"])
    return (logits, torch.stack(streams)) if return_layers else logits
