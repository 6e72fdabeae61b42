"""Small Nuvezen configurations and model folders for the tests, with weights scaled so that the
mechanisms show: sharp attention (a window that is one key off or a lost sink moves the logits), units
whose halves reach their bounds, routers whose choices are clear."""
from __future__ import annotations

import functools
import json
import os
import random
import tempfile
from typing import Dict, Sequence

import numpy as np
import torch

import plain_nuvezen as plain


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, limit=1.5, experts=5, top=3, shared=40, shared_limit=0.75):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared, "limit": shared_limit}
    return out


def latent(heads=3, dim=16, rot_dim=8, vdim=24, rank=40, q_rank=28, window=21, base=3000.0, scale=0.3, mlp=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale,
             "rot": {"dims": rot_dim, "base": base}}
    if window:
        mixer["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def again(layers, index):
    """The entry of a layer that runs layer `index`'s tensors."""
    return {**layers[index], "weights_of": index}


def config(layers, width=72, vocab=211, eps=3e-6):
    return {"architecture": "Nuvezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# Sizes that share nothing: a layer without a feed-forward, a mixture without a shared unit, a shared unit
# whose size is no multiple of the experts', layers that run another's tensors (one of them through a
# third), windows of different lengths.
_A, _B = latent(mlp=moe()), latent(heads=5, dim=12, rot_dim=6, vdim=10, rank=33, q_rank=19, window=17, base=700.0, scale=0.4, mlp=dense())
_C, _D = latent(heads=2, dim=8, rot_dim=12, vdim=20, rank=24, q_rank=45, window=30, scale=0.35), \
    latent(heads=4, dim=10, rot_dim=4, vdim=16, rank=48, q_rank=30, window=9, scale=0.5,
           mlp=moe(ff=16, limit=0.5, experts=4, top=1, shared=0))
MIXED = config([_B, _A, {**_B, "weights_of": 0}, _C, _D, {**_B, "weights_of": 2}, {**_A, "weights_of": 1}])
# Sizes the tensor-core products take.
_E = latent(heads=4, dim=64, rot_dim=32, vdim=64, rank=128, q_rank=112, window=70, base=10000.0, scale=0.12,
            mlp=moe(ff=64, limit=2.5, experts=8, top=2, shared=128, shared_limit=1.25))
WIDE = config([_E, latent(heads=8, dim=32, rot_dim=16, vdim=48, rank=96, q_rank=64, window=50, base=20000.0, scale=0.15, mlp=dense(512)),
               {**_E, "weights_of": 0},
               latent(heads=2, dim=32, rot_dim=64, vdim=128, rank=160, q_rank=96, window=33, base=500.0, scale=0.12,
                      mlp=moe(ff=48, limit=1.0, experts=16, top=4, shared=32, shared_limit=3.0))],
              width=256, vocab=640, eps=2e-5)
# Values the others make equal, even or absent: a width that is no multiple of 8, one head, a window of one
# key (a token sees itself only) and one longer than any request, a rotation of two values, every expert
# chosen, one expert, ranks that are no multiples of 8, rank larger than the heads' values, an unrotated
# part shorter than the rotated one, a layer that runs a later layer's tensors.
_F = latent(heads=6, dim=4, rot_dim=2, vdim=3, rank=33, q_rank=5, window=2, scale=1.0, mlp=moe(ff=8, limit=4.0, experts=2, top=1, shared=7))
ODD = config([{**_F, "weights_of": 3},
              latent(heads=1, dim=6, rot_dim=10, vdim=7, rank=19, q_rank=1, window=1, scale=0.7, mlp=moe(ff=9, experts=1, top=1, shared=5)),
              latent(heads=1, dim=5, rot_dim=10, vdim=9, rank=18, q_rank=21, window=1000, scale=0.7,
                     mlp=moe(ff=12, experts=3, top=3, shared=12, limit=0.25)),
              _F, latent(heads=3, dim=9, rot_dim=14, vdim=2, rank=10, q_rank=90, window=9, scale=0.8, mlp=dense(17))],
             width=100, vocab=97, eps=1e-4)
# A larger one for long steps: many experts, more heads, a latent that is no multiple of 16, no window in
# one layer.
_G = latent(heads=8, dim=32, rot_dim=16, vdim=48, rank=136, q_rank=104, window=90, base=20000.0, scale=0.11,
            mlp=moe(ff=112, limit=2.0, experts=30, top=6, shared=160, shared_limit=1.0))
LARGE = config([_G, latent(heads=16, dim=16, rot_dim=32, vdim=32, rank=256, q_rank=80, window=0, base=20000.0, scale=0.15, mlp=dense(640)),
                {**_G, "weights_of": 0},
                latent(heads=24, dim=24, rot_dim=8, vdim=16, rank=72, q_rank=200, window=200, base=900.0, scale=0.2,
                       mlp=moe(ff=48, limit=1.0, experts=6, top=2, shared=48, shared_limit=2.0))],
               width=384, vocab=1000, eps=1e-5)
ONLY_LATENT = config([latent()])
ONLY_DENSE = config([latent(heads=1, dim=4, rot_dim=2, vdim=4, rank=8, q_rank=8, window=3, mlp=dense(56))])
ONLY_MOE = config([latent(heads=1, dim=4, rot_dim=2, vdim=4, rank=8, q_rank=8, window=3, mlp=moe(ff=32, experts=9, top=3))])
ONLY_AGAIN = config([_B, {**_B, "weights_of": 0}, {**_B, "weights_of": 0}])
# No mask anywhere: a key counts however far back it lies.
FAR = config([latent(window=0, mlp=dense()), latent(heads=5, dim=12, rot_dim=6, vdim=10, rank=33, window=0, mlp=moe())])

CONFIGS = {"mixed": MIXED, "wide": WIDE, "odd": ODD, "large": LARGE, "latent": ONLY_LATENT, "dense": ONLY_DENSE,
           "moe": ONLY_MOE, "again": ONLY_AGAIN, "far": FAR}

# How stored tensors are multiplied (and shifted, where a pair says so), by the end of their names.
SHARP = {"embed": 10.0, ".norm1": 15.0, ".norm2": 15.0, "final.norm": 15.0, ".mix.uq": 25.0, ".mix.dkv": 4.0, ".mix.uk": 4.0,
         ".mix.uv": 10.0, ".mix.sink": (2.0, 5.0), ".mlp.router": 8.0, ".up": 20.0, ".gate": 20.0, ".sg": 20.0}
MILD = {**SHARP, ".mix.uq": 12.0, ".mix.dkv": 2.5, ".mix.uk": 3.0, ".up": 12.0, ".gate": 12.0}
PALE = {"embed": 20.0, ".norm1": 15.0, ".norm2": 15.0}
RULES = {"sharp": SHARP, "mild": MILD, "pale": PALE}


@functools.lru_cache(maxsize=None)
def folder(name: str, store_dtype: str = "float32", seed: int = 7, scaling: str = "sharp") -> str:
    """A model folder of configuration `name` with seeded random weights, scaled."""
    import vipera_rs_b200  # noqa: F401
    from safetensors.torch import load_file, save_file
    from vipera_rs_b200.engine import write_random_model

    path = tempfile.mkdtemp(prefix=f"vipera_nuvezen_{name}_{store_dtype}_{scaling}_")
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
    """A configuration whose sizes, order of layers and constants are drawn from `seed`: windows shorter than
    a page and longer than a request, layers without masks, ranks that are no multiples of 8, mixtures
    with and without shared units, layers without a feed-forward, layers that run others' tensors."""
    rng = random.Random(1000 + seed)
    width = rng.choice([64, 96, 128, 200, 256])
    layers = []
    for _ in range(rng.randint(2, 4)):
        kind = rng.choice(["dense", "moe", "moe", None])
        mlp = None
        if kind == "dense":
            mlp = dense(rng.choice([24, 40, 64, 136]))
        elif kind == "moe":
            experts, ff = rng.choice([1, 2, 5, 8, 19]), rng.choice([8, 16, 24, 64])
            mlp = moe(ff=ff, limit=rng.choice([0.5, 1.0, 3.0, 7.0]), experts=experts, top=rng.randint(1, min(experts, 4)),
                      shared=rng.choice([0, ff // 2, ff, 2 * ff + 8]), shared_limit=rng.choice([0.5, 2.0]))
        dim, rot_dim = rng.choice([8, 16, 24, 32, 64, 128]), rng.choice([2, 8, 16, 32, 64])
        layers.append(latent(heads=rng.choice([1, 2, 3, 8, 16, 17]), dim=dim, rot_dim=rot_dim, vdim=rng.choice([8, 24, 64, 80]),
                             rank=rng.choice([16, 19, 64, 96, 136, 200]), q_rank=rng.choice([8, 31, 64, 96, 160]),
                             window=rng.choice([0, 1, 5, 33, 64, 65, 100, 500]), base=rng.choice([100.0, 10000.0, 500000.0]),
                             scale=(dim + rot_dim) ** -0.5, mlp=mlp))
    own = len(layers)
    for _ in range(rng.choice([0, 1, 3])):
        layers.append(again(layers, rng.randrange(own)))
    return config(layers, width=width, vocab=rng.randint(50, 600), eps=rng.choice([1e-5, 1e-6, 3e-4]))


for _seed in range(16):
    CONFIGS[f"drawn{_seed}"] = drawn(_seed)
