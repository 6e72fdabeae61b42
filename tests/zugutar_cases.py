"""Small Zugutar configurations and model folders for the tests, with weights scaled so that the mechanisms
show: sharp attention (a lost sink, a query's factor that is one position off or a far key moves the logits),
decays held near one (a token counts hundreds of tokens later), routers whose choices are clear."""
from __future__ import annotations

import functools
import json
import os
import random
import tempfile
from typing import Dict, Sequence

import numpy as np
import torch

import plain_zugutar as plain


def moe(ff=24, experts=5, top=2, shared=40):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def attention(heads=6, kv_heads=2, dim=16, vdim=24, scale=0.3, coef=0.7, every=13, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "q_temp": {"coef": coef, "every": every}}, "mlp": mlp}


def parallel(heads=4, kv_heads=2, dim=24, vdim=16, rot=12, base=3000.0, scale=0.25, m_heads=6, m_vdim=20, state=24, groups=3,
             taps=4, norm_groups=5, mlp=None):
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": rot, "base": base}},
        "right": {"heads": m_heads, "vdim": m_vdim, "state": state, "groups": groups, "conv": taps, "norm_groups": norm_groups}},
        "mlp": mlp}


def config(layers, width=72, vocab=211, eps=3e-6, logit_scale=1.5, loop=None):
    out = {"architecture": "Zugutar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}
    if loop:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


# Sizes that share nothing: layers without a feed-forward, a mixture without a shared unit, a shared unit whose
# size is no multiple of the experts', a loop of three passes that begins with either mixer.
MIXED = config([parallel(mlp=moe()), attention(mlp=moe(ff=16, experts=4, top=1, shared=0)),
                parallel(heads=3, kv_heads=3, dim=10, vdim=14, rot=10, base=700.0, scale=0.35, m_heads=4, m_vdim=9, state=40, groups=1,
                         taps=3, norm_groups=2),
                attention(heads=5, kv_heads=1, dim=12, vdim=8, scale=0.4, coef=0.4, every=29, mlp=moe(ff=40, experts=3, top=3, shared=24))],
               loop=(1, 3, 3))
# Sizes the tensor-core products and attention kernels take.
WIDE = config([attention(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.13, coef=0.3, every=50, mlp=moe(ff=64, experts=8, top=2, shared=128)),
               parallel(heads=4, kv_heads=1, dim=64, vdim=64, rot=64, base=10000.0, scale=0.12, m_heads=8, m_vdim=64, state=64, groups=2,
                        taps=4, norm_groups=2, mlp=moe(ff=48, experts=16, top=4, shared=32)),
               parallel(heads=2, kv_heads=2, dim=128, vdim=128, rot=64, base=20000.0, scale=0.09, m_heads=4, m_vdim=32, state=128,
                        groups=1, taps=2, norm_groups=4, mlp=moe(ff=64, experts=4, top=2, shared=0))],
              width=256, vocab=640, eps=2e-5, logit_scale=0.75, loop=(1, 2, 2))
# Values the others make equal, even or absent: a width that is no multiple of 8, one head, one key head, keys
# shorter and longer than values, a factor that changes at every position and one that never does, a rotation of
# two values, one tap, more taps than a short portion has tokens, one state, one value, a norm part per value
# group of odd size, one expert, every expert chosen, a single pass, a negative logit scale.
ODD = config([attention(heads=1, kv_heads=1, dim=5, vdim=9, scale=0.7, coef=1.1, every=1, mlp=moe(ff=9, experts=1, top=1, shared=5)),
              parallel(heads=6, kv_heads=3, dim=7, vdim=3, rot=2, base=50.0, scale=1.0, m_heads=1, m_vdim=21, state=1, groups=1, taps=1,
                       norm_groups=7, mlp=moe(ff=8, experts=2, top=1, shared=7)),
              parallel(heads=1, kv_heads=1, dim=6, vdim=11, rot=6, base=900.0, scale=0.6, m_heads=3, m_vdim=1, state=5, groups=3, taps=11,
                       norm_groups=1),
              parallel(heads=2, kv_heads=1, dim=18, vdim=5, rot=4, scale=0.4, m_heads=2, m_vdim=70, state=19, groups=2, taps=2,
                       norm_groups=20, mlp=moe(ff=12, experts=3, top=3, shared=12)),
              attention(heads=3, kv_heads=3, dim=9, vdim=2, scale=0.8, coef=0.6, every=5000)],
             width=100, vocab=97, eps=1e-4, logit_scale=-2.5, loop=(0, 5, 1))
# A larger one for long steps: more heads, several heads of a group to a block.
LARGE = config([parallel(heads=8, kv_heads=2, dim=128, vdim=128, rot=128, base=20000.0, scale=0.09, m_heads=16, m_vdim=64, state=96,
                         groups=2, taps=4, norm_groups=4, mlp=moe(ff=112, experts=12, top=3, shared=160)),
                attention(heads=8, kv_heads=4, dim=64, vdim=64, scale=0.12, coef=0.2, every=200, mlp=moe(ff=48, experts=6, top=2, shared=48)),
                parallel(heads=3, kv_heads=1, dim=40, vdim=72, rot=24, base=900.0, scale=0.15, m_heads=8, m_vdim=48, state=200, groups=1,
                         taps=5, norm_groups=8, mlp=moe(ff=64, experts=4, top=1, shared=0))],
               width=384, vocab=1000, eps=1e-5, logit_scale=2.5, loop=(0, 2, 2))
ONLY_ATTENTION = config([attention()])
ONLY_PARALLEL = config([parallel()])
ONLY_MOE = config([attention(heads=1, kv_heads=1, dim=4, vdim=4, mlp=moe(ff=32, experts=9, top=3))])
ONLY_LOOP = config([attention(), parallel(mlp=moe())], loop=(0, 2, 4))
# A token counts however far back it lies, through either kind of attention or through the recurrence.
FAR = config([attention(mlp=moe()), parallel()])

CONFIGS = {"mixed": MIXED, "wide": WIDE, "odd": ODD, "large": LARGE, "attention": ONLY_ATTENTION, "parallel": ONLY_PARALLEL,
           "moe": ONLY_MOE, "loop": ONLY_LOOP, "far": FAR}

# How stored tensors are multiplied (and shifted, where a pair says so), by the end of their names.  The step
# sizes' bias is shifted down and the rates are low: a state keeps most of itself over a hundred tokens.
SLOW = {".dt_bias": (30.0, -3.0), ".A_log": (1.0, -2.0), ".right.D": (1.0, 0.3), ".conv": 2.0, ".right.in": 10.0}
SHARP = {"embed": 15.0, ".norm1": 15.0, "final.norm": 15.0, ".mix.q": 15.0, ".mix.k": 20.0, ".mix.v": 8.0, ".mix.g": 15.0,
         ".left.q": 8.0, ".left.k": 8.0, ".left.q.norm": 1.7, ".left.k.norm": 1.7, ".left.v": 8.0, ".left.g": 15.0, ".mlp.router": 14.0,
         ".up": 12.0, ".gate": 12.0, ".sg": 20.0, **SLOW}
MILD = {**SHARP, ".mix.q": 8.0, ".mix.k": 8.0, ".left.q.norm": 1.2, ".left.k.norm": 1.2, ".up": 8.0, ".gate": 8.0}
SOFT = {**MILD, ".mix.q": 5.0, ".mix.k": 5.0, ".left.q": 5.0, ".left.k": 5.0, ".left.q.norm": 1.0, ".left.k.norm": 1.0, ".up": 6.0,
        ".gate": 6.0, ".right.in": 5.0}
PALE = {"embed": 20.0, ".norm1": 15.0, ".dt_bias": (20.0, -1.0), ".mlp.router": 8.0}
RULES = {"sharp": SHARP, "mild": MILD, "soft": SOFT, "pale": PALE}


@functools.lru_cache(maxsize=None)
def folder(name: str, store_dtype: str = "float32", seed: int = 7, scaling: str = "sharp") -> str:
    """A model folder of configuration `name` with seeded random weights, scaled."""
    import vipera_rs_b200  # noqa: F401
    from safetensors.torch import load_file, save_file
    from vipera_rs_b200.engine import write_random_model

    path = tempfile.mkdtemp(prefix=f"vipera_zugutar_{name}_{store_dtype}_{scaling}_")
    write_random_model(path, CONFIGS[name], seed, store_dtype)
    file = os.path.join(path, "model.safetensors")
    tensors = load_file(file)
    for tensor_name in list(tensors):
        for ending, factor in RULES[scaling].items():
            if tensor_name.endswith(ending):
                value = tensors[tensor_name]
                times, plus = factor if isinstance(factor, tuple) else (factor, 0.0)
                tensors[tensor_name] = (value.to(torch.float32) * times + plus).to(value.dtype)
    save_file(tensors, file)
    return path


def read(path: str):
    from safetensors.torch import load_file

    with open(os.path.join(path, "config.json")) as handle:
        return json.load(handle), load_file(os.path.join(path, "model.safetensors"))


_PLAIN: Dict[tuple, tuple] = {}


def _plain(path: str, tokens: Sequence[int]) -> tuple:
    key = (path, tuple(tokens))
    if key not in _PLAIN:
        config, weights = read(path)
        margins = []
        logits = plain.forward(config, weights, list(tokens), margins=margins).numpy()
        least = torch.stack(margins).min(dim=0).values.numpy() if margins else np.full(len(tokens), np.inf)
        _PLAIN[key] = (logits, least)
    return _PLAIN[key]


def plain_logits(path: str, tokens: Sequence[int]) -> np.ndarray:
    return _plain(path, tokens)[0]


def plain_margins(path: str, tokens: Sequence[int]) -> np.ndarray:
    """Per position, the least margin of any router's choice (plain.route)."""
    return _plain(path, tokens)[1]


def drawn(seed: int) -> dict:
    """A configuration whose sizes, order of layers and constants are drawn from `seed`."""
    rng = random.Random(2000 + seed)
    layers = []
    for _ in range(rng.randint(2, 4)):
        mlp = None
        if rng.random() < 0.8:
            experts, ff = rng.choice([1, 2, 5, 8, 19]), rng.choice([8, 16, 24, 64])
            mlp = moe(ff=ff, experts=experts, top=rng.randint(1, min(experts, 4)), shared=rng.choice([0, ff // 2, ff, 2 * ff + 8]))
        kv_heads = rng.choice([1, 2, 3])
        dim = rng.choice([8, 24, 64, 96, 128, 160])
        sizes = dict(kv_heads=kv_heads, heads=kv_heads * rng.choice([1, 2, 5]), dim=dim, vdim=rng.choice([dim, dim, 8, 40, 128]),
                     scale=rng.choice([0.6, 1.0, 1.4]) * dim ** -0.5)
        if rng.random() < 0.45:
            layers.append(attention(coef=rng.choice([0.1, 0.5, 1.0]), every=rng.choice([1, 7, 33, 64, 100, 1000]), mlp=mlp, **sizes))
        else:
            groups, m_vdim = rng.choice([1, 2, 4]), rng.choice([8, 20, 32, 64, 72, 128])
            m_heads = groups * rng.choice([1, 2, 3])
            layers.append(parallel(rot=rng.choice([2, dim // 2, dim]), base=rng.choice([100.0, 10000.0, 500000.0]), m_heads=m_heads,
                                   m_vdim=m_vdim, state=rng.choice([3, 16, 32, 80, 128]), groups=groups, taps=rng.choice([1, 2, 3, 4, 6]),
                                   norm_groups=rng.choice([1, 2, 4, m_heads]) if m_vdim % 4 == 0 else m_heads, mlp=mlp, **sizes))
    start = rng.randint(0, len(layers) - 1)
    loop = rng.choice([None, (start, rng.randint(start + 1, len(layers)), rng.choice([1, 2, 3]))])
    return config(layers, width=rng.choice([64, 96, 128, 200, 256]), vocab=rng.randint(50, 600), eps=rng.choice([1e-5, 1e-6, 3e-4]),
                  logit_scale=rng.choice([1.0, 0.5, 3.0]), loop=loop)


for _seed in range(16):
    CONFIGS[f"drawn{_seed}"] = drawn(_seed)
