"""The kernels' options that Nuvezen brought, each alone against a plain 64-bit restatement of the same
operation: branches that join the stream with the next norms, the query latent's norm beside the cache
write, attention over latents with sinks and with splits that cover a window only (far into a long
history), and the mixture of bounded units chosen by logits beside a gated shared unit in its three
forms; the parallel arrangement beside one that settles what is pending."""
import pytest
import torch

from test_kernels_gpu import _ops, _rel

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


@pytest.mark.parametrize("rows,hidden", [(1, 72), (3, 37), (5, 4096), (2, 5000), (4, 2051), (300, 384), (7, 1536)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_branches_join_the_stream_and_two_norms_follow(rows, hidden, dtype):
    """One and two branches, of several parts, with scales and without; no branch, no norm, one norm, two
    norms with an eps each; rows picked for a last reader, which leaves the stream as it is.  Widths
    with and without whole vectors, short enough for registers and not."""
    ops = _ops()
    g = torch.Generator().manual_seed(rows * 7 + hidden)
    x0 = torch.randn(rows, hidden, generator=g)
    a, b = torch.randn(rows, 1, hidden, generator=g), torch.randn(rows, 5, hidden, generator=g)
    sa, sb = torch.randn(hidden, generator=g), torch.randn(hidden, generator=g)
    g1, g2 = torch.randn(hidden, generator=g), torch.randn(hidden, generator=g)
    eps1, eps2 = 1e-5, 0.3
    limit = 2e-6 if dtype == torch.float32 else 5e-3

    def norm(x, gain, eps):
        return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain.double()

    both = x0.double() + sa.double() * a.double().sum(1) + sb.double() * b.double().sum(1)
    for branches, want in (([(a, 1, sa), (b, 5, sb)], both), ([(b, 5, None)], x0.double() + b.double().sum(1)), ([], x0.double())):
        on_device = [(v.reshape(rows, -1).to(DEV), parts, None if s is None else s.to(DEV)) for v, parts, s in branches]
        for norms in (2, 1, 0):
            if not norms and not branches:
                continue
            x = x0.to(DEV)
            outs = [torch.full((rows, hidden), float("nan"), dtype=dtype, device=DEV) for _ in range(norms)]
            ops.join_norms(x, on_device, [(gain.to(DEV), eps, out) for (gain, eps), out in zip(((g1, eps1), (g2, eps2)), outs)])
            assert _rel(x.cpu(), want) < 2e-6
            for (gain, eps), out in zip(((g1, eps1), (g2, eps2)), outs):
                assert _rel(out.float().cpu(), norm(want, gain, eps)) < limit
        picked = torch.tensor([rows - 1, 0, rows // 2], dtype=torch.int32)
        x, out = x0.to(DEV), torch.full((3, hidden), float("nan"), dtype=dtype, device=DEV)
        ops.join_norms(x, on_device, [(g1.to(DEV), eps1, out)], rows=picked.to(DEV))
        assert torch.equal(x.cpu(), x0)
        assert _rel(out.float().cpu(), norm(want[picked.long()], g1, eps1)) < limit


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("q_rank,rank,rot,own", [(28, 40, 8, True), (1, 19, 10, True), (300, 512, 64, True), (96, 64, 2, False)])
def test_the_query_latent_is_normed_beside_the_cache_write(q_rank, rank, rot, own, dtype):
    ops = _ops()
    g = torch.Generator().manual_seed(q_rank)
    page, entries = 8, [(0, 11), (21, 2), (5, 1)]
    entry = torch.tensor([e for e, (_, n) in enumerate(entries) for _ in range(n)], dtype=torch.int32)
    position = torch.tensor([first + i for first, n in entries for i in range(n)], dtype=torch.int32)
    tokens, start = len(entry), 3
    proj = torch.randn(tokens, start + q_rank + rank + rot + 5, generator=g)
    cq_off, kv_off = start, start + q_rank
    wq, wk = 1 + 0.3 * torch.randn(q_rank, generator=g), 1 + 0.3 * torch.randn(rank, generator=g)
    angle = torch.arange(32, dtype=torch.float64)[:, None] * 50.0 ** (-torch.arange(rot // 2, dtype=torch.float64) / (rot // 2))
    table = torch.tensor([[4, 1, -1], [0, 7, 2], [5, -1, -1]], dtype=torch.int32)
    k_pool = torch.full((9, page, 1, rank), float("nan"), dtype=dtype, device=DEV)
    v_pool = torch.full((9, page, 1, rot), float("nan"), dtype=dtype, device=DEV)
    cq = torch.full((tokens, q_rank), float("nan"), dtype=dtype, device=DEV)
    eps = 0.02
    ops.latent_store(proj.to(DEV), kv_off=kv_off if own else -1, norm_weight=wk.to(DEV), eps=eps, positions=position.to(DEV),
                     token_entry=entry.to(DEV), block_table=table.to(DEV), cos=angle.cos().float().to(DEV),
                     sin=angle.sin().float().to(DEV), k_pool=k_pool, v_pool=v_pool, rot_dim=rot, cq_off=cq_off,
                     cq_norm_weight=wq.to(DEV), cq=cq)
    limit = 2e-6 if dtype == torch.float32 else 5e-3

    def norm(x, w):
        return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w.double()

    assert _rel(cq.float().cpu(), norm(proj[:, cq_off:cq_off + q_rank].double(), wq)) < limit
    if not own:
        assert torch.isnan(k_pool.float()).all() and torch.isnan(v_pool.float()).all()
        return
    latent = norm(proj[:, kv_off:kv_off + rank].double(), wk)
    raw = proj[:, kv_off + rank:kv_off + rank + rot].double()
    written = torch.zeros(9, page, dtype=torch.bool)
    for t in range(tokens):
        p = int(position[t])
        at = int(table[int(entry[t]), p // page]), p % page
        written[at] = True
        assert _rel(k_pool[at].float().cpu().view(-1), latent[t]) < limit
        u, v, c, s = raw[t, 0::2], raw[t, 1::2], angle[p].cos(), angle[p].sin()
        turned = torch.stack([u * c - v * s, v * c + u * s], dim=-1).reshape(-1)
        assert _rel(v_pool[at].float().cpu().view(-1), turned) < limit
    assert torch.isnan(k_pool.float().cpu()[~written]).all()     # nothing else was touched


# heads, unrotated, rotated, value size, rank; the window; per request (tokens already in the cache, tokens of the step)
FOLDS = {
    "prompts": ((12, 32, 64, 32, 512), 100, [(0, 37), (130, 5), (64, 1), (15, 18)]),
    "decode": ((12, 32, 64, 32, 512), 300, [(1700, 1), (63, 1), (0, 1), (2029, 1), (64, 1), (2048 + 300, 1)]),
    "far_decode": ((4, 16, 8, 16, 64), 72, [(5000, 1), (4095, 1), (71, 1), (72, 1), (3967, 1)]),
    "one_key": ((3, 16, 8, 8, 40), 1, [(900, 1), (0, 2), (127, 3)]),
    "many_heads": ((20, 8, 24, 16, 136), 65, [(1000, 3), (300, 1), (0, 9)]),
    "long_prompts": ((3, 16, 8, 8, 40), 130, [(0, 903), (400, 450)]),
    "one_head": ((1, 16, 16, 16, 96), 48, [(2000, 40), (63, 66), (640, 1)]),
    "no_window": ((4, 16, 16, 16, 200), 0, [(0, 70), (345, 7), (200, 1)]),
    "plain_sizes": ((5, 12, 6, 10, 33), 40, [(500, 1), (0, 45), (39, 2)]),
}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("form", ["whole", "cut", "head_major"])
@pytest.mark.parametrize("name", sorted(FOLDS))
def test_attention_over_latents_with_sinks_and_a_window(name, form, dtype):
    """Queries apart from the projection, sinks from far below to far above the scores, requests of
    unequal history in one step, pages in a shuffled order; the pages a window has left are marked as
    given back and hold nothing that may be read."""
    ops = _ops()
    (heads, d, rot, dv, rank), window, requests = FOLDS[name]
    tensor_cores = dtype == torch.bfloat16 and rank % 8 == 0 and rot % 8 == 0
    if form != "whole" and not tensor_cores:
        pytest.skip("one form only")
    if form == "head_major" and d % 8:
        pytest.skip("the grouped products take heads of whole vectors")
    page = 16
    g = torch.Generator().manual_seed(5)
    lengths = [before + new for before, new in requests]
    width_pages = max(-(-n // page) for n in lengths)
    table = torch.full((len(requests), width_pages), -1, dtype=torch.int32)
    needed = [(e, i) for e, (before, new) in enumerate(requests) for i in range(-(-lengths[e] // page))
              if not window or (i + 1) * page > before - window + 1]
    order = torch.randperm(len(needed) + 3, generator=g).tolist()
    for (e, i), physical in zip(needed, order):
        table[e, i] = physical
    k_pool = torch.randn(len(order), page, 1, rank, generator=g).to(dtype)
    v_pool = torch.randn(len(order), page, 1, rot, generator=g).to(dtype)
    spare = sorted(set(range(len(order))) - {int(p) for p in table.flatten() if p >= 0})
    k_pool[spare], v_pool[spare] = float("nan"), float("nan")
    entry = [e for e, (_, new) in enumerate(requests) for _ in range(new)]
    position = [before + i for before, new in requests for i in range(new)]
    tokens = len(entry)
    q = torch.randn(tokens, heads * (d + rot), generator=g)
    up_k = (torch.randn(heads * d, rank, generator=g) * 0.3).to(dtype)
    up_v = (torch.randn(heads, rank, dv, generator=g) * 0.1).to(dtype)
    sink = torch.linspace(-120.0, 6.0, heads) if heads > 1 else torch.tensor([1.5])
    if heads > 2:
        sink[1], sink[2] = 120.0, 1.0       # all of the weight goes to the sink; a share of it does
    scale = 0.12
    angle = torch.arange(max(lengths) + 1, dtype=torch.float64)[:, None] * (100.0 ** (-torch.arange(rot // 2, dtype=torch.float64) / (rot // 2)))
    cos, sin = angle.cos(), angle.sin()
    want = torch.zeros(tokens, heads * dv, dtype=torch.float64)
    qd = q.double().view(tokens, heads, d + rot)
    for t in range(tokens):
        p, e = position[t], entry[t]
        first = max(0, p - window + 1) if window else 0
        slots = [int(table[e, j // page]) * page + j % page for j in range(first, p + 1)]
        c, kr = k_pool.view(-1, rank)[slots].double(), v_pool.view(-1, rot)[slots].double()
        u, v = qd[t, :, d::2], qd[t, :, d + 1::2]
        turned = torch.stack([u * cos[p] - v * sin[p], v * cos[p] + u * sin[p]], dim=-1).reshape(heads, rot)
        absorbed = torch.einsum("hdr,hd->hr", up_k.double().view(heads, d, rank), qd[t, :, :d])
        scores = torch.cat([scale * (absorbed @ c.T + turned @ kr.T), sink.double()[:, None]], dim=1)
        weights = torch.softmax(scores, dim=1)[:, :-1]
        want[t] = torch.einsum("hrv,hr->hv", up_v.double(), weights @ c).reshape(-1)
    qa = torch.full((tokens, heads, rank + rot), float("nan"), device=DEV)
    mixed = torch.full((tokens, heads, rank), float("nan"), device=DEV)
    out = torch.full((tokens, heads * dv), float("nan"), dtype=dtype, device=DEV)
    max_keys = max(lengths)
    single = all(new == 1 for _, new in requests)
    floats = ops.latent_part_floats(tokens, heads, rank, rot, max_keys, ops.sm_count(torch.device(DEV)), window, single)
    splits = ops.latent_plan(tokens, heads, rank, rot, max_keys, ops.sm_count(torch.device(DEV)), window, single)[3]
    if window:      # the splits are no more than the window needs, whatever the history
        assert splits * ops.latent_plan(tokens, heads, rank, rot, max_keys, ops.sm_count(torch.device(DEV)), window, single)[2] <= window + 256
    part = torch.full((floats,), float("nan"), device=DEV) if form != "whole" and floats else None
    buffers = None
    if form == "head_major":
        padded = -(-tokens // 128) * 128

        def scratch(rows, columns, kind):
            return torch.full((rows, columns), float("nan") if kind != torch.int32 else -1, dtype=kind, device=DEV)

        buffers = {"padded": padded, "up_k_t": up_k.view(heads, d, rank).transpose(1, 2).contiguous().to(DEV),
                   "up_v_rows": up_v.transpose(1, 2).contiguous().to(DEV),
                   "a_heads": scratch(heads * padded, d, torch.bfloat16), "qa_heads": scratch(heads * padded, rank, torch.float32),
                   "q_rot": scratch(tokens, heads * rot, torch.float32), "l_heads": scratch(heads * padded, rank, torch.bfloat16),
                   "o_heads": scratch(heads * padded, dv, torch.float32),
                   "tile_group": scratch(1, heads * padded // 128, torch.int32).view(-1)}
    proj = torch.full((tokens, 8), float("nan"), device=DEV)       # holds nothing this call may read
    ops.latent_attention(proj, q_off=0, g_off=-1, kv_off=-1, up_k=up_k.to(DEV), up_v=up_v.to(DEV), norm_weight=None, eps=1e-6,
                         positions=torch.tensor(position, dtype=torch.int32, device=DEV),
                         token_entry=torch.tensor(entry, dtype=torch.int32, device=DEV), block_table=table.to(DEV),
                         cos=cos.float().to(DEV), sin=sin.float().to(DEV), k_pool=k_pool.to(DEV), v_pool=v_pool.to(DEV), qa=qa,
                         latent_out=mixed, out=out, heads=heads, head_dim=d, rot_dim=rot, value_dim=dv, scale=scale,
                         max_keys=max_keys, part=part, head_major=buffers, window=window, sink=sink.to(DEV), q=q.to(DEV), single=single)
    ops.check_kernel_status(torch.device(DEV))
    got = out.cpu().double()
    assert torch.isfinite(got).all()
    assert float((got - want).abs().max()) <= (2e-5 if dtype == torch.float32 else 2e-2) * float(want.abs().max())


def _mixture_reference(h, router, gate_row, gate, up, down, top, always, limits, slope):
    """64-bit: choice by the logits, weights the softmax over the chosen; the last `always` units count for
    all tokens with the sigmoid of the gate's row; bounded units."""
    logits = h.double() @ router.double().T
    ranked = logits.sort(dim=-1, descending=True)
    chosen, weights = ranked.indices[:, :top], torch.softmax(ranked.values[:, :top], dim=-1)
    margin = ranked.values[:, top - 1] - ranked.values[:, top] if top < logits.shape[1] else torch.full((h.shape[0],), 1.0)
    shared = torch.sigmoid(h.double() @ gate_row.double()) if gate_row is not None else torch.ones(h.shape[0], dtype=torch.float64)
    every = []
    for e in range(gate.shape[0]):
        a = torch.clamp(h.double() @ gate[e].double().T, max=limits[e])
        b = torch.clamp(h.double() @ up[e].double().T, -limits[e], limits[e])
        every.append((a * torch.sigmoid(slope * a) * (b + 1)) @ down[e].double().T)
    every = torch.stack(every, dim=1)
    real = gate.shape[0] - always
    out = (weights[:, :, None] * torch.gather(every[:, :real], 1, chosen[:, :, None].expand(-1, -1, h.shape[1]))).sum(1)
    return out + shared[:, None] * every[:, real:].sum(1), chosen, weights, shared, margin


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("gated_shared", [True, False])
@pytest.mark.parametrize("tokens,hidden,ff,experts,always,top,tile_rows", [
    (5, 64, 32, 6, 2, 3, 8),         # few assignments: tiles of 8 rows
    (9, 37, 13, 4, 1, 1, 8),         # the same with rows that are no whole vectors
    (300, 128, 64, 12, 1, 4, 128),   # bfloat16: grouped tensor-core products; 32-bit: tiles of 32 rows
    (70, 72, 24, 5, 0, 2, 32),       # an inner size the tensor-core form refuses; no shared unit
    (200, 256, 48, 3, 3, 3, 128),    # every expert chosen
    (700, 64, 208, 40, 2, 6, 128),   # more experts than tiles of rows
])
def test_mixture_of_bounded_units_chosen_by_logits(tokens, hidden, ff, experts, always, top, tile_rows, gated_shared, dtype):
    ops = _ops()
    if gated_shared and not always:
        pytest.skip("no shared unit to gate")
    g = torch.Generator().manual_seed(tokens + hidden)
    matrices, slope = experts + always, 1.702
    h = torch.randn(tokens, hidden, generator=g).to(dtype)
    router = torch.randn(experts, hidden, generator=g) * 4.0     # logits far apart: their softmax over all would underflow
    gate_row = torch.randn(hidden, generator=g) * 0.2 if gated_shared else None
    gate, up = ((torch.randn(matrices, ff, hidden, generator=g) * 0.2).to(dtype) for _ in range(2))
    down = (torch.randn(matrices, hidden, ff, generator=g) * 0.2).to(dtype)
    limits = [0.5 + 0.25 * (e % 7) for e in range(experts)] + [3.0 - 0.5 * e for e in range(always)]
    want, want_chosen, want_weight, shared, margin = _mixture_reference(
        h.float(), router, gate_row, gate.float(), up.float(), down.float(), top, always, limits, slope)
    slots = top + always
    chosen = torch.full((tokens, slots), -7, dtype=torch.int32, device=DEV)
    weight = torch.full((tokens, slots), float("nan"), device=DEV)
    scratch = torch.zeros(ops.moe_scratch_words(tokens, slots, matrices), dtype=torch.int32, device=DEV)
    capacity = ops.moe_capacity(tokens, slots, matrices)
    act = torch.full((capacity, ff), float("nan"), dtype=dtype, device=DEV)
    rows = torch.full((tokens, slots * hidden), float("nan"), device=DEV)
    xs = torch.full((capacity, hidden), float("nan"), dtype=dtype, device=DEV)
    ys = torch.full((capacity, hidden), float("nan"), device=DEV)
    gate_group = ops.MOE_GATE_GROUP if dtype == torch.bfloat16 and ff % ops.MOE_GATE_GROUP == 0 else ff
    gate_up = torch.stack([gate.view(matrices, ff // gate_group, gate_group, hidden),
                           up.view(matrices, ff // gate_group, gate_group, hidden)], dim=2).reshape(matrices, 2 * ff, hidden)
    expected_rows = 32 if dtype == torch.float32 and tile_rows == 128 else tile_rows
    assert ops.moe_form(tokens, slots, hidden, ff, gate_group, dtype)[0] == expected_rows
    table = router if gate_row is None else torch.cat([router, gate_row[None]])
    ops.moe(h.to(DEV), router=table.to(DEV), gate_up=gate_up.contiguous().to(DEV), down=down.to(DEV), gate_group=gate_group, top=top,
            groups=1, keep=1, group_top=1, softmax_scores=False, renormalize=False, activation=ops.ACT_CLAMPED, chosen=chosen,
            weight=weight, scratch=scratch, act=act, rows=rows, xs=xs, ys=ys, always=always, logit_scores=True,
            always_gate=gated_shared, unit_limit=torch.tensor(limits, device=DEV), unit_slope=slope)
    ops.check_kernel_status(torch.device(DEV))
    got = rows.view(tokens, slots, hidden).double().sum(1).cpu()
    assert torch.isfinite(got).all()
    clear = margin > 1e-3      # (a choice that hangs on the last bits may come out either way)
    assert clear.float().mean() > 0.95
    assert (chosen[:, :top].cpu().long() == want_chosen)[clear].all()
    assert torch.allclose(weight[:, :top].double().cpu()[clear], want_weight[clear], rtol=1e-4, atol=1e-6)
    assert torch.allclose(weight[:, top:].double().cpu(), shared[:, None].expand(-1, always), rtol=1e-5, atol=1e-7)
    assert _rel(got[clear], want[clear]) < (2e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_arrangement_beside_one_that_settles_what_is_pending(dtype):
    """Parallel layers and pre-norm layers take turns in one model: a pre-norm layer finds the stream
    complete, whoever ran before it; and the parallel arrangement without scales."""
    import numpy as np

    import nuvezen_cases as cases
    from vipera_rs_b200.config import architecture_of
    from vipera_rs_b200.config.spec import LayerSpec, ScheduleEntry
    from vipera_rs_b200.cache import CachePools
    from vipera_rs_b200.engine.loader import build_kernels
    from vipera_rs_b200.engine.runner import ModelRunner, StepInput
    from vipera_rs_b200.parts.model import DecoderModel, model_schema
    from vipera_rs_b200.weights import RandomSource
    import dataclasses

    import plain_nuvezen as plain

    arch = architecture_of(cases.ONLY_DENSE)
    spec = arch.model_spec(arch.config_from_dict(cases.config([cases.latent(mlp=cases.dense())] * 4)))
    layers = []
    for index, layer in enumerate(spec.layers):
        block = "prenorm" if index in (1, 2) else "parallel"
        layers.append(LayerSpec(block, layer.prefix, layer.parts, layer.names, {"hidden_size": spec.hidden_size}))
    spec = dataclasses.replace(spec, layers=layers, schedule=[ScheduleEntry(i, i) for i in range(4)])
    run = torch.float32 if dtype == "float32" else torch.bfloat16
    source = RandomSource(model_schema(spec), 3, run)
    model = DecoderModel(spec, source, run, DEV)
    build_kernels(model.kernel_families())
    pools = CachePools(model.cache_requests, page_size=16, num_pages=4, num_state_slots=1, dtype=run, device=torch.device(DEV))
    runner = ModelRunner(model, pools, max_model_len=64)
    tokens = list(range(5, 45))
    pools.manager.open(0)
    pools.manager.reserve(0, 40)
    got = runner.run(StepInput(requests=[0], tokens=np.asarray(tokens, dtype=np.int32), counts=[40], pos0=[0], fresh=[1],
                               logit_rows=np.arange(40, dtype=np.int32))).double().cpu()
    w = {name[:-len(".weight")] if name.endswith(".weight") else name: source.get(name) for name in source.names()}
    eps, mixer = 3e-6, cases.latent()["mixer"]
    x = w["embed"].double()[torch.tensor(tokens)]
    for i in range(4):
        def n(stream, which, i=i):
            return plain.zero_centred_norm(stream, w[f"l{i}.{which}"], eps)
        if i in (1, 2):
            x = x + plain.latent_attention(n(x, "norm1"), w, f"l{i}.mix", mixer, eps)
            x = x + plain.dense_ff(n(x, "norm2"), w, f"l{i}.mlp")
        else:
            x = x + plain.latent_attention(n(x, "norm1"), w, f"l{i}.mix", mixer, eps) + plain.dense_ff(n(x, "norm2"), w, f"l{i}.mlp")
    want = plain.zero_centred_norm(x, w["final.norm"], eps) @ w["embed"].double().T
    assert _rel(got, want) < (1e-5 if dtype == "float32" else 4e-2)
