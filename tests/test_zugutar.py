"""Zugutar without a GPU: configuration, order of layer runs, tensor names, what the layers keep between
steps, and the plain implementation against other ways of writing its mechanisms; what the tests' sharpened
weights make visible (the sink, the query's factor, gates, norms, the passes of a loop, a far token)."""
import copy
import json

import numpy as np
import pytest
import torch

import helpers
import plain_zugutar as plain
import zugutar_cases as cases
import vipera_rs_b200  # noqa: F401
from vipera_rs_b200 import errors
from vipera_rs_b200.cache.pools import plan_groups
from vipera_rs_b200.config import architecture_of
from vipera_rs_b200.engine.planner import plan_memory, spec_cache_requests
from vipera_rs_b200.parts.attention import GQAttention
from vipera_rs_b200.parts.base import CacheBundle, FixedState, PagedKV
from vipera_rs_b200.parts.rotary import QueryFactor

F = torch.float64


def spec_of(name):
    arch = architecture_of(cases.CONFIGS[name])
    return arch, arch.model_spec(arch.config_from_dict(cases.CONFIGS[name]))


def test_configuration_reads_back_and_refuses_what_it_does_not_know():
    arch, spec = spec_of("mixed")
    for name in cases.CONFIGS:
        config = arch.config_from_dict(cases.CONFIGS[name])
        assert arch.config_from_dict(config.to_dict()) == config
    assert spec.head_name is None and spec.logit_scale == 1.5 and spec.final_norm.params["weight_offset"] == 1.0
    # three passes over layers 1 and 2, each with caches of its own; the embedding's rows join before two of them
    assert [(e.layer, e.cache, e.adds_embedding) for e in spec.schedule] == [
        (0, 0, False), (1, 1, False), (2, 2, False), (1, 3, True), (2, 4, False), (1, 5, True), (2, 6, False), (3, 7, False)]
    assert [sorted(layer.parts) for layer in spec.layers] == [["ffn", "mixer", "mixer_norm"]] * 2 + [["mixer", "mixer_norm"]] + \
        [["ffn", "mixer", "mixer_norm"]]
    (left_name, left, left_scale), (right_name, right, right_scale) = spec.layers[0].parts["mixer"].params["branches"]
    assert (left_name, left_scale, right_name, right_scale) == ("left", 0.5, "right", 0.5)
    assert (left.params["head_norm"], left.params["sink"], left.params["output_gate"]) == (True, True, "heads")
    assert left.params["position"].params["rotary_dims"] == 12 and left.params["position"].params["exact_angles"] is True
    assert (right.kind, right.params["groups"], right.params["norm_groups"], right.params["taps"]) == ("mamba2", 3, 5, 4)
    ffn = spec.layers[0].parts["ffn"].params
    assert (ffn["weight_on"], ffn["score"], ffn["shared_size"], ffn["shared_gate"]) == ("input", "sigmoid", 40, True)
    assert not spec.layers[1].parts["ffn"].params.get("shared_size")
    single = spec_of("odd")[1]
    assert len(single.schedule) == 5 and not any(e.adds_embedding for e in single.schedule)   # one pass
    for path, value, error in ((("layers", 0, "type"), "mamba2", errors.UnsupportedError),
                               (("layers", 1, "mixer", "kv_heads"), 4, errors.InvalidArgumentError),
                               (("layers", 1, "mixer", "q_temp", "every"), 0, errors.InvalidArgumentError),
                               (("layers", 1, "mixer", "q_temp"), {"coef": 1.0}, errors.UnsupportedError),
                               (("layers", 0, "mixer", "left", "rot", "dims"), 26, errors.InvalidArgumentError),
                               (("layers", 0, "mixer", "left", "rot", "dims"), 11, errors.InvalidArgumentError),
                               (("layers", 0, "mixer", "right", "groups"), 4, errors.InvalidArgumentError),
                               (("layers", 0, "mixer", "right", "norm_groups"), 7, errors.InvalidArgumentError),
                               (("layers", 0, "mixer", "right", "conv"), 0, errors.InvalidArgumentError),
                               (("layers", 0, "mlp", "router", "top"), 6, errors.InvalidArgumentError),
                               (("layers", 0, "mlp", "kind"), "dense", errors.UnsupportedError),
                               (("loop", "stop"), 5, errors.InvalidArgumentError),
                               (("loop", "times"), 0, errors.InvalidArgumentError)):
        bad = json.loads(json.dumps(cases.MIXED))
        at = bad
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(error):
            arch.config_from_dict(bad)
    assert arch.config_from_dict(json.loads(json.dumps({k: v for k, v in cases.MIXED.items() if k != "loop"}))).layer_runs() == [(i, False) for i in range(4)]


def test_tensor_names_of_a_written_folder():
    _, weights = cases.read(cases.folder("mixed", "bfloat16", scaling="pale"))
    names = set(weights)
    assert {"embed", "final.norm", "l0.norm1", "l0.mix.left.q", "l0.mix.left.k", "l0.mix.left.v", "l0.mix.left.q.norm",
            "l0.mix.left.k.norm", "l0.mix.left.g", "l0.mix.left.o", "l0.mix.left.out", "l0.mix.right.out", "l0.mix.right.in",
            "l0.mix.right.conv", "l0.mix.right.conv.b", "l0.mix.right.dt_bias", "l0.mix.right.A_log", "l0.mix.right.D",
            "l0.mix.right.norm", "l0.mix.right.o", "l1.mix.q", "l1.mix.g", "l1.mix.o", "l0.mlp.router", "l0.mlp.e4.down",
            "l0.mlp.shared.sg", "l0.mlp.shared.up", "l3.mlp.e2.gate"} <= names
    assert not {"head", "l0.norm2", "l1.mix.q.norm", "l1.mlp.shared.up", "l2.mlp.router", "l0.mix.left.sink"} & names
    shape = {name: tuple(weights[name].shape) for name in names}
    assert shape["l0.mix.right.in"] == (2 * 120 + 2 * 3 * 24 + 6, 72) and shape["l0.mix.right.conv"] == (120 + 144, 4)
    assert shape["l0.mix.left.g"] == (4, 72) and shape["l1.mix.g"] == (6 * 24, 72) and shape["l0.mix.left.q.norm"] == (24,)
    assert shape["l0.mix.left.out"] == (72,) and shape["l0.mlp.shared.sg"] == (1, 72)
    assert weights["l0.norm1"].abs().max() < 1.0      # stored around zero


def test_what_layers_keep_between_steps():
    _, spec = spec_of("mixed")
    requests = spec_cache_requests(spec)
    first = CacheBundle.of(left=PagedKV(2, 64, None),      # heads filled up to a tile
                           right=CacheBundle.of(conv=FixedState((3, 264)), scan=FixedState((6 * 24 * 20,))))
    again = CacheBundle.of(left=PagedKV(3, 64, None),
                           right=CacheBundle.of(conv=FixedState((2, 36 + 80)), scan=FixedState((4 * 40 * 9,))))
    assert requests[0] == first and requests[1] == requests[3] == requests[5] == PagedKV(2, 64, None)
    assert requests[2] == requests[4] == requests[6] == again and requests[7] == PagedKV(1, 64, None)
    groups, states = plan_groups(requests)
    assert sorted(len(group.slots) for group in groups) == [1, 3, 4] and len(states) == 8
    assert spec_cache_requests(spec_of("odd")[1])[1].members[1][1] == CacheBundle.of(scan=FixedState((21,)))   # one tap keeps nothing
    assert plan_memory(spec, 256, 4, "bfloat16", device_bytes=10**9)["feasible"]
    # up to 64 values, up to 128, and heads no tile holds
    sizes = [GQAttention._stored_sizes({"head_dim": d, "value_dim": dv, "tile_heads": True})
             for d, dv in ((64, 64), (5, 9), (65, 8), (40, 72), (128, 128), (160, 8))]
    assert sizes == [(64, 64), (64, 64), (128, 128), (128, 128), (128, 128), (160, 8)]
    assert GQAttention._stored_sizes({"head_dim": 40}) == (40, 40)


@pytest.mark.parametrize("coef,every", [(0.7, 13), (0.5, 1), (0.3, 5000), (1.2, 3), (0.25, 7.5)])
def test_the_query_factor_steps_at_whole_multiples(coef, every):
    table = QueryFactor({"coef": coef, "every": every}, 4000, "cpu").table().double()
    want = plain.temperature(4000, {"coef": coef, "every": every})
    assert torch.allclose(table, want, rtol=1e-7, atol=0)
    steps = [p for p in range(1, 100) if want[p] != want[p - 1]]
    assert steps == [p for p in range(1, 100) if int((p + 1) // every) != int(p // every)]    # position p counts p + 1 tokens
    small = QueryFactor({"coef": coef, "every": every}, 4000, "cpu")
    small.prepare(10)
    assert small.table().numel() == 10
    small.prepare(50)
    assert small.table().numel() == 50 and torch.equal(small.table().double(), table[:50])


def test_the_sink_is_one_more_score_of_zero():
    torch.manual_seed(3)
    scores = torch.randn(3, 6, 6, dtype=F) * 4 - 2
    got = plain.causal_softmax(scores, sink=True)
    seen = torch.tril(torch.ones(6, 6, dtype=torch.bool))
    padded = torch.cat([scores.masked_fill(~seen, float("-inf")), torch.zeros(3, 6, 1, dtype=F)], dim=-1)
    assert torch.allclose(got, torch.softmax(padded, dim=-1)[..., :6], atol=1e-14) and (got.sum(-1) < 1).all()
    assert torch.allclose(plain.causal_softmax(scores).sum(-1), torch.ones(3, 6, dtype=F))


def test_the_recurrence_against_its_unrolled_sum_and_its_chunks():
    """y_t = sum_{s <= t} exp(l_t - l_s) dt_s (c_t . b_s) x_s + d x_t with l the running sum of log decays: the
    form the chunked kernels use, also from a chunk's starting state on."""
    torch.manual_seed(4)
    count, heads, n, size = 37, 3, 5, 4
    x, b, c = (torch.randn(count, heads, k, dtype=F) for k in (size, n, n))
    dt, rate, d = torch.rand(count, heads, dtype=F), torch.rand(heads, dtype=F), torch.randn(heads, dtype=F)
    want = plain.state_recurrence(x, b, c, dt, rate, d)
    logs = torch.cumsum(-rate * dt, dim=0)
    weights = torch.exp(logs[:, None] - logs[None, :]) * dt[None] * torch.einsum("thn,shn->tsh", c, b)
    weights = weights * torch.tril(torch.ones(count, count, dtype=F))[:, :, None]
    assert torch.allclose(torch.einsum("tsh,shp->thp", weights, x) + d[:, None] * x, want, atol=1e-10)
    state, out = torch.zeros(heads, n, size, dtype=F), []
    for begin in range(0, count, 16):
        end = min(begin + 16, count)
        l = torch.cumsum(-rate * dt[begin:end], dim=0)
        part = plain.state_recurrence(x[begin:end], b[begin:end], c[begin:end], dt[begin:end], rate, d)
        out.append(part + torch.exp(l)[:, :, None] * torch.einsum("hnp,thn->thp", state, c[begin:end]))
        left = torch.exp(l[-1][None] - l) * dt[begin:end]
        state = torch.exp(l[-1])[:, None, None] * state + torch.einsum("th,thn,thp->hnp", left, b[begin:end], x[begin:end])
    assert torch.allclose(torch.cat(out), want, atol=1e-10)


def test_the_convolution_against_torch():
    torch.manual_seed(5)
    x, weight, bias = torch.randn(20, 6, dtype=F), torch.randn(6, 4, dtype=F), torch.randn(6, dtype=F)
    padded = torch.nn.functional.pad(x.T[None], (3, 0))
    want = torch.nn.functional.conv1d(padded, weight[:, None], bias, groups=6)[0].T
    assert torch.allclose(plain.causal_conv(x, weight, bias), want, atol=1e-12)


def test_a_weight_on_the_input_is_not_one_on_the_output():
    torch.manual_seed(2)
    h = torch.randn(9, 24, dtype=F)
    w = {"e.gate": torch.randn(40, 24, dtype=F), "e.up": torch.randn(40, 24, dtype=F), "e.down": torch.randn(24, 40, dtype=F)}
    inside, outside = plain.unit(0.3 * h, w, "e"), 0.3 * plain.unit(h, w, "e")
    assert (inside - outside).abs().max() > 0.1 * outside.abs().max()
    # both halves of the unit see it: the product of two linear maps, one through silu
    gate, up = 0.3 * plain.product(h, w["e.gate"]), 0.3 * plain.product(h, w["e.up"])
    assert torch.allclose(plain.product(plain.silu(gate) * up, w["e.down"]), inside)


def _logits(name, tokens, change=None, scaling="sharp"):
    config, weights = cases.read(cases.folder(name, "float32", scaling=scaling))
    config, weights = copy.deepcopy(config), dict(weights)
    if change is not None:
        change(config, weights)
    return plain.forward(config, weights, tokens).numpy()


def test_what_the_sharpened_weights_make_visible(monkeypatch):
    """The GPU tests rest on this: with the tests' weights a mechanism that is left out or one position off
    moves the logits by far more than the tolerances."""
    tokens = helpers.random_tokens(cases.MIXED["vocab"], 80, 5)
    want = _logits("mixed", tokens)
    scale = np.abs(want).max()

    def moved(change, rows=slice(40, None)):
        return float(np.abs(_logits("mixed", tokens, change)[rows] - want[rows]).max() / scale)

    def set_to(name, value):
        def change(config, weights):
            weights[name] = torch.full_like(weights[name], value)
        return change

    for name, value in (("l0.norm1", 0.0), ("l0.mix.left.q.norm", 1.0), ("l0.mix.left.k.norm", 1.0), ("l0.mix.left.g", 0.0),
                        ("l1.mix.g", 0.0), ("l0.mix.left.out", 1.1), ("l0.mix.right.out", 1.1), ("l0.mix.right.D", 0.0),
                        ("l0.mix.right.dt_bias", 0.0), ("l0.mix.right.A_log", -20.0), ("l0.mix.right.conv.b", 0.3),
                        ("l0.mix.right.norm", 1.2), ("l0.mlp.shared.sg", 0.0), ("final.norm", 0.0)):
        assert moved(set_to(name, value)) > 0.005, name

    def mixer(layer, *path_value):
        def change(config, weights):
            at = config["layers"][layer]["mixer"]
            for key in path_value[:-2]:
                at = at[key]
            at[path_value[-2]] = path_value[-1]
        return change

    for change in (mixer(1, "q_temp", "every", 14), mixer(1, "q_temp", "every", 12), mixer(1, "q_temp", "coef", 0.6),
                   mixer(0, "left", "rot", "dims", 14), mixer(0, "left", "rot", "base", 2000.0),
                   mixer(0, "left", "scale", 0.3), mixer(0, "right", "norm_groups", 6)):
        assert moved(change, slice(0, None)) > 0.003

    def one_pass_less(config, weights):
        config["loop"]["times"] = 2
    assert moved(one_pass_less) > 0.05

    for function, other in (("temperature", lambda count, m: torch.cat([torch.ones(1, dtype=F), plain_temperature(count, m)[:-1]])),
                            ("layer_runs", lambda config: [(i, False) for i, _ in plain_runs(config)]),
                            ("causal_softmax", lambda scores, sink=False: plain_softmax(scores, False))):
        plain_temperature, plain_runs, plain_softmax = plain.temperature, plain.layer_runs, plain.causal_softmax
        with monkeypatch.context() as patch:
            patch.setattr(plain, function, other)
            assert moved(None) > 0.005, function

    # a token counts however far back it lies
    tokens = helpers.random_tokens(cases.FAR["vocab"], 330, 6)
    changed = list(tokens)
    changed[3] = (changed[3] + 1) % cases.FAR["vocab"]
    a, b = _logits("far", tokens), _logits("far", changed)
    assert np.abs(a[-20:] - b[-20:]).max() / np.abs(a).max() > 2e-3
    # and through the recurrence alone
    for name in ("l1.mix.left.o", "l0.mix.o"):
        def without(config, weights, name=name):
            weights[name] = torch.zeros_like(weights[name])
        a, b = _logits("far", tokens, without), _logits("far", changed, without)
        assert np.abs(a[-20:] - b[-20:]).max() / np.abs(a).max() > 1e-3, name
