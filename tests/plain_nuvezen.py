"""A plain, slow implementation of the Nuvezen decoder in float64: one function per mechanism, whole
sequences at once, no code shared with the package.

``weights`` maps the names of the design's own weight file (``embed``, ``l0.mix.uq``,
``l1.mlp.e3.up``, ...) to tensors; ``config`` is the design's config.json as a dict.

Notation.  The stream starts as ``x = E[token]``; a layer computes both of its branches from the same x,

    x += s1 * mixer(N1(x)) + s2 * ff(N2(x))      (without the second term where it has no feed-forward)

with s1, s2 a number per channel and N(x) = x / rms(x) * (1 + w); the logits are ``E N(x)``.  A layer
may run another layer's tensors.  Mixer: attention whose queries come through a normed latent and whose
keys and values are products of a normed latent, with one rotated key part (pairs ``(2i, 2i + 1)``)
shared by the heads, a window, and a softmax whose denominator also holds ``exp(sink_h)``.
Feed-forwards: a gated unit with silu; or a mixture of clamped gated units chosen by router logits,
weighted by the softmax of the chosen logits, beside a gated shared unit.
"""
import torch

F = torch.float64


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def zero_centred_norm(x, w, eps):
    """The stored weight is the gain's distance from one."""
    return rms_norm(x, 1.0 + w.to(F), eps)


def rotate_interleaved(x, positions, rot):
    """x [T, ..., d]: values (2i, 2i + 1) of the first rot.dims turn by position * base^(-2i/dims)."""
    dims = int(rot["dims"])
    frequency = float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=F) / dims)
    angle = positions.to(F)[:, None] * frequency[None, :]
    cos, sin = torch.cos(angle), torch.sin(angle)
    while cos.dim() < x.dim():
        cos, sin = cos.unsqueeze(1), sin.unsqueeze(1)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def visible(count, mask):
    """visible[i, j]: 0 <= i - j < mask.size (every j <= i without a mask)."""
    i = torch.arange(count)[:, None]
    j = torch.arange(count)[None, :]
    seen = j <= i
    if mask is not None:
        seen = seen & (i - j < int(mask["size"]))
    return seen


def softmax_with_sink(scores, seen, sink):
    """scores [H, T, T]; the denominator also holds exp(sink_h), a term that stands for no token."""
    scores = scores.masked_fill(~seen, float("-inf"))
    sink = sink.to(F)[:, None, None]
    top = torch.maximum(scores.max(dim=-1, keepdim=True).values, sink)
    weights = torch.exp(scores - top)
    return weights / (weights.sum(-1, keepdim=True) + torch.exp(sink - top))


def queries(h, w, prefix, mixer, eps):
    """[T, heads, dim + rot_dim], through the normed query latent."""
    latent = rms_norm(h @ w[f"{prefix}.dq"].to(F).T, w[f"{prefix}.dq.norm"].to(F), eps)
    q = latent @ w[f"{prefix}.uq"].to(F).T
    return q.reshape(h.shape[0], int(mixer["heads"]), int(mixer["dim"]) + int(mixer["rot_dim"]))


def latent_attention(h, w, prefix, mixer, eps):
    heads, d, dv, rank = (int(mixer[k]) for k in ("heads", "dim", "vdim", "kv_rank"))
    count = h.shape[0]
    positions = torch.arange(count)
    q = queries(h, w, prefix, mixer, eps)
    down = h @ w[f"{prefix}.dkv"].to(F).T
    latent = rms_norm(down[:, :rank], w[f"{prefix}.dkv.norm"].to(F), eps)
    key_rot = rotate_interleaved(down[:, rank:], positions, mixer["rot"])
    q_rot = rotate_interleaved(q[..., d:], positions, mixer["rot"])
    key = (latent @ w[f"{prefix}.uk"].to(F).T).reshape(count, heads, d)
    value = (latent @ w[f"{prefix}.uv"].to(F).T).reshape(count, heads, dv)
    scores = torch.einsum("ihd,jhd->hij", q[..., :d], key) + torch.einsum("ihd,jd->hij", q_rot, key_rot)
    weights = softmax_with_sink(scores * float(mixer["scale"]), visible(count, mixer.get("mask")), w[f"{prefix}.sink"])
    out = torch.einsum("hij,jhd->ihd", weights, value).reshape(count, heads * dv)
    return out @ w[f"{prefix}.o"].to(F).T


def dense_ff(h, w, prefix):
    gate = h @ w[f"{prefix}.gate"].to(F).T
    return (gate * torch.sigmoid(gate) * (h @ w[f"{prefix}.up"].to(F).T)) @ w[f"{prefix}.down"].to(F).T


def clamped_unit(h, w, prefix, limit):
    """g s(1.702 g) (u + 1), g bounded above by the limit and u on both sides."""
    gate = torch.clamp(h @ w[f"{prefix}.gate"].to(F).T, max=float(limit))
    up = torch.clamp(h @ w[f"{prefix}.up"].to(F).T, -float(limit), float(limit))
    return (gate * torch.sigmoid(1.702 * gate) * (up + 1.0)) @ w[f"{prefix}.down"].to(F).T


def route(h, w, prefix, router):
    """(chosen [T, top], weights [T, top], margin [T]): the largest logits, weighted by the softmax over
    themselves.  The margin is the gap between the last chosen logit and the best one left out."""
    top = int(router["top"])
    ranked = (h @ w[f"{prefix}.router"].to(F).T).sort(dim=-1, descending=True)
    margin = ranked.values[:, top - 1] - ranked.values[:, top] if top < ranked.values.shape[1] else \
        torch.full((h.shape[0],), float("inf"), dtype=F)
    return ranked.indices[:, :top], torch.softmax(ranked.values[:, :top], dim=-1), margin


def mixture(h, w, prefix, mlp, margins=None):
    chosen, weights, margin = route(h, w, prefix, mlp["router"])
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        tokens, places = torch.where(chosen == e)
        if tokens.numel():
            out[tokens] += weights[tokens, places][:, None] * clamped_unit(h[tokens], w, f"{prefix}.e{e}", mlp["expert"]["limit"])
    if mlp.get("shared") is not None:
        gate = torch.sigmoid(h @ w[f"{prefix}.shared.sg"].to(F).T)
        out = out + gate * clamped_unit(h, w, f"{prefix}.shared", mlp["shared"]["limit"])
    return out


def tensors_of(layers, index):
    """The layer whose tensors layer `index` runs."""
    while layers[index].get("weights_of") is not None:
        index = int(layers[index]["weights_of"])
    return index


def forward(config, weights, tokens, return_layers=False, margins=None):
    """Logits [T, vocab] of one sequence; with `return_layers` also the stream after every layer.  A list
    given as `margins` receives every router's margin [T]."""
    w = weights
    eps = float(config["norm"]["eps"])
    x = w["embed"].to(F)[torch.tensor(tokens)]
    streams = []
    for index, layer in enumerate(config["layers"]):
        if layer["type"] != "latent_attention":
            raise ValueError(layer["type"])
        p = f"l{tensors_of(config['layers'], index)}"
        mixed = latent_attention(zero_centred_norm(x, w[f"{p}.norm1"], eps), w, f"{p}.mix", layer["mixer"], eps)
        total = w[f"{p}.ls1"].to(F) * mixed
        mlp = layer.get("mlp")
        if mlp is not None:
            h = zero_centred_norm(x, w[f"{p}.norm2"], eps)
            out = dense_ff(h, w, f"{p}.mlp") if mlp["kind"] == "dense" else mixture(h, w, f"{p}.mlp", mlp, margins)
            total = total + w[f"{p}.ls2"].to(F) * out
        x = x + total
        streams.append(x.clone())
    logits = zero_centred_norm(x, w["final.norm"], eps) @ w["embed"].to(F).T
    return (logits, torch.stack(streams)) if return_layers else logits
