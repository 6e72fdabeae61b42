"""Nuvezen without a GPU: configuration, tensor names, layers that run others' tensors, what the layers
keep between steps, and the plain implementation against other ways of writing its mechanisms; what the
tests' sharpened weights make visible (a window's edge, the sink, the bounds, the scales, a far key)."""
import copy
import json

import numpy as np
import pytest
import torch

import helpers
import nuvezen_cases as cases
import plain_nuvezen as plain
import vipera_rs_b200  # noqa: F401
from vipera_rs_b200 import errors
from vipera_rs_b200.cache.pools import plan_groups
from vipera_rs_b200.config import architecture_of
from vipera_rs_b200.engine.planner import plan_memory, spec_cache_requests
from vipera_rs_b200.parts.base import PagedKV

F = torch.float64


def spec_of(name):
    arch = architecture_of(cases.CONFIGS[name])
    return arch, arch.model_spec(arch.config_from_dict(cases.CONFIGS[name]))


def test_configuration_reads_back_and_refuses_what_it_does_not_know():
    arch, spec = spec_of("mixed")
    config = arch.config_from_dict(cases.MIXED)
    assert arch.config_from_dict(config.to_dict()) == config
    assert spec.head_name is None and spec.final_norm.params["weight_offset"] == 1.0
    # four layers with tensors of their own; the others run theirs, each with a cache of its own
    assert [layer.prefix for layer in spec.layers] == ["l0", "l1", "l3", "l4"]
    assert [(e.layer, e.cache, e.writes_cache) for e in spec.schedule] == [
        (0, 0, True), (1, 1, True), (0, 2, True), (2, 3, True), (3, 4, True), (0, 5, True), (1, 6, True)]
    assert [sorted(layer.parts) for layer in spec.layers][2] == ["mixer", "mixer_norm"]
    mixer, ffn = spec.layers[1].parts["mixer"].params, spec.layers[1].parts["ffn"].params
    assert (mixer["q_rank"], mixer["sink"], mixer["window"], mixer["position"].kind) == (28, "learned", 21, "rope_interleaved")
    assert mixer["position"].params["exact_angles"] is True
    assert (ffn["score"], ffn["limit"], ffn["shared_limit"], ffn["shared_size"], ffn["shared_gate"]) == ("logit", 1.5, 0.75, 40, True)
    assert not spec.layers[3].parts["ffn"].params.get("shared_size")
    # a layer may run the tensors of a layer that comes later
    _, odd = spec_of("odd")
    assert [layer.prefix for layer in odd.layers] == ["l1", "l2", "l3", "l4"] and odd.schedule[0].layer == 2
    for path, value, error in ((("layers", 0, "type"), "attention", errors.UnsupportedError),
                               (("layers", 3, "mixer", "rot", "dims"), 10, errors.InvalidArgumentError),   # not the rotated part
                               (("layers", 1, "mlp", "router", "top"), 6, errors.InvalidArgumentError),
                               (("layers", 1, "mlp", "kind"), "sparse", errors.UnsupportedError),
                               (("layers", 1, "mlp", "expert"), {"ff": 24}, errors.UnsupportedError),      # without its limit
                               (("layers", 2, "weights_of"), 9, errors.InvalidArgumentError),
                               (("layers", 0, "weights_of"), 2, errors.InvalidArgumentError),              # a circle
                               (("layers", 2, "weights_of"), 1, errors.InvalidArgumentError),              # other sizes
                               (("layers", 2, "mixer", "mask", "size"), 18, errors.InvalidArgumentError)):
        bad = json.loads(json.dumps(cases.MIXED))      # (no entry shares another's dictionaries)
        at = bad
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(error):
            arch.config_from_dict(bad)


def test_tensor_names_of_a_written_folder():
    path = cases.folder("mixed", "bfloat16", scaling="pale")
    _, weights = cases.read(path)
    names = set(weights)
    assert {"embed", "final.norm", "l0.norm1", "l0.norm2", "l0.ls1", "l0.ls2", "l0.mix.dq", "l0.mix.dq.norm", "l0.mix.uq",
            "l0.mix.dkv", "l0.mix.dkv.norm", "l0.mix.uk", "l0.mix.uv", "l0.mix.sink", "l0.mix.o", "l0.mlp.gate", "l0.mlp.up",
            "l0.mlp.down", "l1.mlp.router", "l1.mlp.e0.gate", "l1.mlp.e4.down", "l1.mlp.shared.gate", "l1.mlp.shared.up",
            "l1.mlp.shared.down", "l1.mlp.shared.sg", "l3.mix.o", "l3.ls1", "l4.mlp.e3.up"} <= names
    assert "head" not in names and "l0.mix.q" not in names and "l4.mlp.shared.up" not in names
    assert "l3.norm2" not in names and "l3.ls2" not in names
    assert not any(name.startswith(("l2.", "l5.", "l6.")) for name in names)     # they run others' tensors
    assert tuple(weights["l1.mix.uq"].shape) == (3 * 24, 28) and tuple(weights["l1.mix.dkv"].shape) == (40 + 8, 72)
    assert tuple(weights["l1.mlp.shared.sg"].shape) == (1, 72) and tuple(weights["l1.mlp.shared.up"].shape) == (40, 72)
    assert weights["l0.norm1"].abs().max() < 1.0      # stored around zero


def test_a_second_branch_that_nothing_reads_is_left_aside():
    arch = architecture_of(cases.MIXED)
    config = arch.config_from_dict(cases.MIXED)
    assert arch.ignorable(config, "l3.norm2.weight") and arch.ignorable(config, "l3.ls2.weight")
    assert not arch.ignorable(config, "l0.norm2.weight") and not arch.ignorable(config, "l3.ls1.weight")
    assert not arch.ignorable(config, "l9.norm2.weight") and not arch.ignorable(config, "l2.norm2.weight")


def test_what_layers_keep_between_steps():
    _, spec = spec_of("mixed")
    requests = spec_cache_requests(spec)
    b = PagedKV(1, 33, 17, value_dim=6)
    assert requests == {0: b, 1: PagedKV(1, 40, 21, value_dim=8), 2: b, 3: PagedKV(1, 24, 30, value_dim=12),
                        4: PagedKV(1, 48, 9, value_dim=4), 5: b, 6: PagedKV(1, 40, 21, value_dim=8)}
    groups, states = plan_groups(requests)
    assert len(groups) == 4 and not states        # layers of one geometry share page numbers, not pages
    assert plan_memory(spec, 256, 4, "bfloat16", device_bytes=10**9)["feasible"]


def test_the_sink_is_one_more_score_without_a_value():
    torch.manual_seed(3)
    scores = torch.randn(3, 5, 5, dtype=F) * 4
    sink = torch.tensor([-2.0, 0.5, 7.0], dtype=F)
    seen = plain.visible(5, {"size": 3})
    got = plain.softmax_with_sink(scores, seen, sink)
    padded = torch.cat([scores.masked_fill(~seen, float("-inf")), sink[:, None, None].expand(3, 5, 1)], dim=-1)
    assert torch.allclose(got, torch.softmax(padded, dim=-1)[..., :5], atol=1e-14)
    assert (got.sum(-1) < 1).all() and got[2].sum(-1).max() < 0.9     # a large sink takes most of the weight
    assert seen.sum(-1).tolist() == [1, 2, 3, 3, 3] and bool(seen[4, 2]) and not bool(seen[4, 1])


def test_latent_attention_with_absorbed_matrices():
    """q . (U c) = (U^T q) . c and sum_j p_j V c_j = V sum_j p_j c_j: the form the kernels use."""
    path = cases.folder("latent", "float32", scaling="mild")
    config, w = cases.read(path)
    mixer, eps = config["layers"][0]["mixer"], config["norm"]["eps"]
    heads, d, dv, rank = (mixer[k] for k in ("heads", "dim", "vdim", "kv_rank"))
    torch.manual_seed(1)
    h = torch.randn(50, config["width"], dtype=F)
    want = plain.latent_attention(h, w, "l0.mix", mixer, eps)
    positions = torch.arange(50)
    cq = h @ w["l0.mix.dq"].to(F).T
    cq = cq / torch.sqrt((cq * cq).mean(-1, keepdim=True) + eps) * w["l0.mix.dq.norm"].to(F)
    q = (cq @ w["l0.mix.uq"].to(F).T).reshape(50, heads, -1)
    down = h @ w["l0.mix.dkv"].to(F).T
    c = plain.rms_norm(down[:, :rank], w["l0.mix.dkv.norm"].to(F), eps)
    kr = plain.rotate_interleaved(down[:, rank:], positions, mixer["rot"])
    qa = torch.einsum("thd,hdr->thr", q[..., :d], w["l0.mix.uk"].to(F).reshape(heads, d, rank))
    scores = torch.einsum("ihr,jr->hij", qa, c) + \
        torch.einsum("ihd,jd->hij", plain.rotate_interleaved(q[..., d:], positions, mixer["rot"]), kr)
    p = plain.softmax_with_sink(scores * mixer["scale"], plain.visible(50, mixer["mask"]), w["l0.mix.sink"])
    out = torch.einsum("hvr,ihr->ihv", w["l0.mix.uv"].to(F).reshape(heads, dv, rank), torch.einsum("hij,jr->ihr", p, c))
    assert torch.allclose(out.reshape(50, -1) @ w["l0.mix.o"].to(F).T, want, atol=1e-9)


def test_a_bounded_unit_is_the_sum_of_its_pieces():
    """The unit is a sum over its inner features, and a feature of zeros gives 0 although the other half
    has one added to it: cut into pieces of another size, the last filled up, the pieces add up."""
    torch.manual_seed(2)
    h = torch.randn(9, 24, dtype=F) * 2
    w = {"s.gate": torch.randn(40, 24, dtype=F), "s.up": torch.randn(40, 24, dtype=F), "s.down": torch.randn(24, 40, dtype=F)}
    whole = plain.clamped_unit(h, w, "s", 1.25)
    gate, up = (torch.cat([w[f"s.{n}"], torch.zeros(8, 24, dtype=F)]) for n in ("gate", "up"))
    down = torch.cat([w["s.down"], torch.zeros(24, 8, dtype=F)], dim=1)
    pieces = sum(plain.clamped_unit(h, {"p.gate": gate[i:i + 16], "p.up": up[i:i + 16], "p.down": down[:, i:i + 16]}, "p", 1.25)
                 for i in range(0, 48, 16))
    assert torch.allclose(pieces, whole, atol=1e-10)
    # the bounds: the gate from above only, the other half on both sides
    eye = {"e.gate": torch.tensor([[1.0, 0.0]], dtype=F), "e.up": torch.tensor([[0.0, 1.0]], dtype=F), "e.down": torch.ones(1, 1, dtype=F)}
    unit = lambda g, u: float(plain.clamped_unit(torch.tensor([[g, u]], dtype=F), eye, "e", 2.0))  # noqa: E731
    assert unit(5.0, 0.3) == unit(2.0, 0.3) and unit(1.0, 9.0) == unit(1.0, 2.0) and unit(1.0, -9.0) == unit(1.0, -2.0)
    assert unit(-5.0, 0.3) != unit(-2.0, 0.3) and unit(1.0, -1.0) == 0.0


def test_the_router_weighs_the_chosen_logits_only():
    torch.manual_seed(5)
    h = torch.randn(50, 16, dtype=F)
    w = {"m.router": torch.randn(6, 16, dtype=F)}
    chosen, weights, margin = plain.route(h, w, "m", {"experts": 6, "top": 2})
    logits = h @ w["m.router"].T
    every = torch.softmax(logits, dim=-1)
    picked = torch.gather(every, 1, chosen)
    # the softmax over all, divided by its sum over the chosen, is the softmax over the chosen
    assert torch.allclose(weights, picked / picked.sum(-1, keepdim=True)) and torch.allclose(weights.sum(-1), torch.ones(50, dtype=F))
    assert torch.equal(chosen, logits.topk(2, dim=-1).indices) and (margin > 0).all()


def _logits(name, tokens, change=None, scaling="sharp"):
    config, weights = cases.read(cases.folder(name, "float32", scaling=scaling))
    config, weights = copy.deepcopy(config), dict(weights)
    if change is not None:
        change(config, weights)
    return plain.forward(config, weights, tokens).numpy()


def test_what_the_sharpened_weights_make_visible():
    """The GPU tests rest on this: with the tests' weights a window that is one key off, a sink, a bound,
    a scale or a gate that is left out and a far key all move the logits by far more than the
    tolerances."""
    tokens = helpers.random_tokens(cases.MIXED["vocab"], 80, 5)
    want = _logits("mixed", tokens)
    scale = np.abs(want).max()

    def moved(change, rows=slice(40, None)):
        return float(np.abs(_logits("mixed", tokens, change)[rows] - want[rows]).max() / scale)

    for layer in range(7):
        for step in (-1, 1):
            def window(config, weights, layer=layer, step=step):
                config["layers"][layer]["mixer"]["mask"]["size"] += step
            assert moved(window) > 0.01, (layer, step)

    def set_to(name, value):
        def change(config, weights):
            weights[name] = torch.full_like(weights[name], value)
        return change

    for name, value in (("l0.mix.sink", -50.0), ("l1.mix.sink", -50.0), ("l0.ls1", 1.0), ("l1.ls2", 1.0), ("l1.mlp.shared.sg", 0.0),
                        ("l0.norm1", 0.0), ("l1.norm2", 0.0)):
        assert moved(set_to(name, value)) > 0.01, name

    def limits(which):
        def change(config, weights):
            for layer in (1, 6):
                config["layers"][layer]["mlp"][which]["limit"] *= 1.3
        return change
    assert moved(limits("expert")) > 0.01 and moved(limits("shared")) > 0.01

    def not_again(config, weights):     # the layer's tensors run once instead of three times
        config["layers"] = [layer for i, layer in enumerate(config["layers"]) if i not in (2, 5)]
        config["layers"][4]["weights_of"] = 1
        for key in list(weights):
            if key.startswith(("l3.", "l4.")):
                weights[f"l{int(key[1]) - 1}{key[2:]}"] = weights[key]
    assert moved(not_again) > 0.05

    # without masks a token counts however far back it lies
    tokens = helpers.random_tokens(cases.FAR["vocab"], 260, 6)
    changed = list(tokens)
    changed[3] = (changed[3] + 1) % cases.FAR["vocab"]
    a, b = _logits("far", tokens), _logits("far", changed)
    assert np.abs(a[-20:] - b[-20:]).max() / np.abs(a).max() > 1e-3
