"""The kernels' options that Zugutar brought, each alone against a plain 64-bit restatement of the same
operation: up to four branches that join the stream, two of them normed on the way; heads with a norm of their
own, rotation and a factor per position; attention with a sink of score 0 and a gate per head or per value;
Mamba-2's recurrence walking and in chunks; the mixture whose weights multiply what the experts read; and the
embedding's rows added again in front of arrangements that settle what is pending."""
import math
import os

import numpy as np
import pytest
import torch

from test_kernels_gpu import _ops, _paged_case, _rel

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F = torch.float64


@pytest.mark.parametrize("rows,hidden", [(1, 72), (3, 37), (5, 4096), (2, 5000), (4, 2051), (300, 384), (7, 1536)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_normed_branches_join_the_stream(rows, hidden, dtype):
    """Two normed branches (one of several parts) beside two plain ones, one normed alone, three and four plain
    ones; with and without norms behind; rows picked for a last reader.  The branches come in any order."""
    ops = _ops()
    g = torch.Generator().manual_seed(rows * 11 + hidden)
    x0 = torch.randn(rows, hidden, generator=g)
    a, b, c, d = (torch.randn(rows, parts, hidden, generator=g) * size for parts, size in ((1, 3.0), (2, 0.02), (5, 1.0), (1, 1.0)))
    sa, sb, sc = (torch.randn(hidden, generator=g) for _ in range(3))
    gain, eps = torch.randn(hidden, generator=g), 0.2
    limit = 2e-6 if dtype == torch.float32 else 5e-3

    def normed(v, scale, e):
        total = v.double().sum(1)
        total = total / torch.sqrt((total * total).mean(-1, keepdim=True) + e)
        return total if scale is None else total * scale.double()

    def plainly(v, scale):
        return v.double().sum(1) if scale is None else v.double().sum(1) * scale.double()

    cases = (([(a, 1, sa, 1e-5), (c, 5, None), (b, 2, sb, 1e-3), (d, 1, sc)], normed(a, sa, 1e-5) + normed(b, sb, 1e-3) + plainly(c, None) + plainly(d, sc)),
             ([(c, 5, sc), (b, 2, None, 1e-4)], plainly(c, sc) + normed(b, None, 1e-4)),
             ([(a, 1, sa, 1e-5)], normed(a, sa, 1e-5)),
             ([(a, 1, sa, 1e-5), (d, 1, None), (c, 5, sb)], normed(a, sa, 1e-5) + plainly(d, None) + plainly(c, sb)),
             ([(a, 1, sa), (b, 2, None), (c, 5, None)], plainly(a, sa) + plainly(b, None) + plainly(c, None)),
             ([(a, 1, sa), (b, 2, sb), (c, 5, sc), (d, 1, None)], plainly(a, sa) + plainly(b, sb) + plainly(c, sc) + plainly(d, None)))
    for branches, added in cases:
        want = x0.double() + added
        on_device = [(v.reshape(rows, -1).to(DEV), parts, None if s is None else s.to(DEV), *rest) for v, parts, s, *rest in branches]
        for norms in (1, 0):
            x = x0.to(DEV)
            out = torch.full((rows, hidden), float("nan"), dtype=dtype, device=DEV)
            ops.join_norms(x, on_device, [(gain.to(DEV), eps, out)] if norms else [])
            assert _rel(x.cpu(), want) < 3e-6
            if norms:
                assert _rel(out.float().cpu(), want / torch.sqrt((want * want).mean(-1, keepdim=True) + eps) * gain.double()) < limit
        picked = torch.tensor([rows - 1, 0, rows // 2], dtype=torch.int32)
        x, out = x0.to(DEV), torch.full((3, hidden), float("nan"), dtype=dtype, device=DEV)
        ops.join_norms(x, on_device, [(gain.to(DEV), eps, out)], rows=picked.to(DEV))
        chosen = want[picked.long()]
        assert torch.equal(x.cpu(), x0)
        assert _rel(out.float().cpu(), chosen / torch.sqrt((chosen * chosen).mean(-1, keepdim=True) + eps) * gain.double()) < limit


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,d,dv,rot,style", [(3, 1, 96, 96, 96, "neox"), (6, 2, 10, 7, 6, "neox"), (5, 5, 128, 64, 64, "interleaved"),
                                                           (1, 1, 256, 3, 2, "neox"), (12, 3, 33, 160, 0, "none"), (2, 1, 64, 64, 62, "neox")])
def test_heads_on_their_way_to_the_cache(heads, kv_heads, d, dv, rot, style, dtype):
    """A norm per head, rotation, a factor per position for queries only; each alone and together; the rows hold
    more than q, k and v; what no token writes stays untouched."""
    ops = _ops()
    g = torch.Generator().manual_seed(d + rot)
    page, entries = 8, [(0, 11), (21, 2), (5, 1)]
    entry = torch.tensor([e for e, (_, n) in enumerate(entries) for _ in range(n)], dtype=torch.int32)
    position = torch.tensor([first + i for first, n in entries for i in range(n)], dtype=torch.int32)
    table = torch.tensor([[4, 1, -1], [0, 7, 2], [5, -1, -1]], dtype=torch.int32)
    tokens, width = len(entry), (heads + kv_heads) * d + kv_heads * dv
    qkv = torch.randn(tokens, width + 5, generator=g)
    wq, wk, eps = 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.3 * torch.randn(d, generator=g), 0.03
    factor = 1 + torch.rand(40, generator=g)
    half = max(rot // 2, 1)
    angle = torch.arange(40, dtype=F)[:, None] * 30.0 ** (-torch.arange(half, dtype=F) / half)
    code = {"neox": ops.ROPE_NEOX, "interleaved": ops.ROPE_INTERLEAVED, "none": ops.ROPE_NONE}[style]
    limit = 2e-6 if dtype == torch.float32 else 5e-3
    for with_norm, with_factor, norm_size in ((True, True, None), (True, False, d - 1 if d > rot else d), (False, True, None)):
        k_pool = torch.full((9, page, kv_heads, d), float("nan"), dtype=dtype, device=DEV)
        v_pool = torch.full((9, page, kv_heads, dv), float("nan"), dtype=dtype, device=DEV)
        q_out = torch.full((tokens, heads * d), float("nan"), dtype=dtype, device=DEV)
        ops.head_rows(qkv.to(DEV), q_out, num_heads=heads, num_kv_heads=kv_heads, head_dim=d, value_dim=dv, rot_dims=rot,
                      positions=position.to(DEV), cos=angle.cos().float().to(DEV), sin=angle.sin().float().to(DEV), style=code,
                      k_pool=k_pool, v_pool=v_pool, token_entry=entry.to(DEV), block_table=table.to(DEV), page_size=page,
                      write_cache=True, q_norm=wq.to(DEV) if with_norm else None, k_norm=wk.to(DEV) if with_norm else None,
                      eps=eps, q_factor=factor.to(DEV) if with_factor else None, norm_size=norm_size)

        def head(rows, weight, t):
            rows = rows.double()
            if with_norm:
                rows = rows / torch.sqrt((rows * rows).sum(-1, keepdim=True) / (norm_size or d) + eps) * weight.double()
            out = rows.clone()
            if style != "none":
                c, s = angle[int(position[t])].cos(), angle[int(position[t])].sin()
                u, v = (slice(0, rot, 2), slice(1, rot, 2)) if style == "interleaved" else (slice(0, half), slice(half, rot))
                out[:, u], out[:, v] = rows[:, u] * c - rows[:, v] * s, rows[:, v] * c + rows[:, u] * s
            return out

        written = torch.zeros(9, page, dtype=torch.bool)
        for t in range(tokens):
            p = int(position[t])
            q = head(qkv[t, :heads * d].view(heads, d), wq, t) * (float(factor[p]) if with_factor else 1.0)
            k = head(qkv[t, heads * d:(heads + kv_heads) * d].view(kv_heads, d), wk, t)
            at = int(table[int(entry[t]), p // page]), p % page
            written[at] = True
            assert _rel(q_out[t].float().cpu().view(heads, d), q) < limit
            assert _rel(k_pool[at].float().cpu(), k) < limit
            assert _rel(v_pool[at].float().cpu(), qkv[t, (heads + kv_heads) * d:width].view(kv_heads, dv).double()) < limit
        assert torch.isnan(k_pool.float().cpu()[~written]).all() and torch.isnan(v_pool.float().cpu()[~written]).all()


@pytest.mark.parametrize("heads,kv_heads,d,page", [(4, 2, 64, 16), (3, 1, 128, 64), (5, 5, 48, 8)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("per_head,with_sink", [(True, True), (False, False), (True, False)])
def test_attention_with_a_gate_per_head(heads, kv_heads, d, page, dtype, per_head, with_sink):
    """The general kernel, the flash kernel's ending, the split-key kernel's combine and its cluster forms; the
    gate sits behind other columns, at an offset no vector starts on where it is one per head."""
    ops = _ops()
    lengths, counts = [70, 200, 131, 64, 5, 300], [70, 67, 1, 2, 5, 1]
    entries = len(lengths)
    lengths, counts, table, k_pool, v_pool, keys, values, q = _paged_case(
        entries, heads, kv_heads, d, page, dtype, seed=heads * 10 + d, lengths=lengths, counts=counts)
    scale, total = 1.0 / math.sqrt(d), sum(counts)
    g = torch.Generator().manual_seed(5)
    offset = 23 if per_head else 24
    wide = torch.randn(total, offset + heads * (1 if per_head else d) + (9 if per_head else 8), generator=g) * 2.0
    gate = wide[:, offset:offset + heads * (1 if per_head else d)].reshape(total, heads, -1).double()
    want = torch.zeros(total, heads, d, dtype=F)
    t = 0
    for e, (n, c) in enumerate(zip(lengths, counts)):
        for i in range(c):
            for h in range(heads):
                k, v = (x[e][:n - c + i + 1, h * kv_heads // heads].double() for x in (keys, values))
                s = (k @ q[t, h].double()) * scale
                s = torch.cat([s, torch.zeros(1, dtype=F)]) if with_sink else s
                want[t, h] = torch.softmax(s, dim=0)[:len(k)] @ v * torch.sigmoid(gate[t, h])
            t += 1
    qd = q.to(dtype).reshape(total, heads * d).to(DEV)
    kp, vp, tb, wide_d = k_pool.to(DEV), v_pool.to(DEV), table.to(DEV), wide.to(DEV)
    position = torch.tensor([p for n, c in zip(lengths, counts) for p in range(n - c, n)], dtype=torch.int32, device=DEV)
    entry = torch.tensor([e for e, c in enumerate(counts) for _ in range(c)], dtype=torch.int32, device=DEV)
    limit = 3e-6 if dtype == torch.float32 else 1e-2
    common = dict(num_heads=heads, num_kv_heads=kv_heads, head_dim=d, scale=scale, sink=with_sink, gate_offset=offset, gate_per_head=per_head)
    out = torch.full_like(qd, float("nan"))
    ops.attention(qd, out, kp, vp, token_seq=entry, positions=position, block_table=tb, gate=wide_d, **common)
    assert _rel(out.float().cpu().view(total, heads, d), want) < limit
    if dtype != torch.bfloat16 or d not in ops.TC_ATTENTION_HEAD_DIMS:
        return
    common["sink_values"] = torch.zeros(heads, device=DEV) if with_sink else None
    starts = torch.tensor(np.concatenate([[0], np.cumsum(counts)]), dtype=torch.int32, device=DEV)
    pos0 = torch.tensor([n - c for n, c in zip(lengths, counts)], dtype=torch.int32, device=DEV)
    out = torch.full_like(qd, float("nan"))
    ops.attention_prefill(qd, out, kp, vp, entry_starts=starts, entry_pos0=pos0, block_table=tb, num_entries=entries, gate=wide_d, **common)
    assert _rel(out.float().cpu().view(total, heads, d), want) < limit
    out = torch.full_like(qd, float("nan"))
    ops.attention_prefill(qd, out, kp, vp, entry_starts=starts, entry_pos0=pos0, block_table=tb, num_entries=entries, gate=wide_d,
                          skip_single=True, **common)
    chunk, splits = ops.decode_splits(entries, kv_heads, 300, ops.sm_count(DEV))
    scratch = torch.full((ops.attention_decode_scratch_floats(entries, heads, d, splits),), float("nan"), device=DEV)
    ops.attention_decode(qd, out, kp, vp, positions=pos0, block_table=tb, window=0, chunk=chunk, num_splits=splits, scratch=scratch,
                         entry_starts=starts, gate=wide_d, **common)
    assert _rel(out.float().cpu().view(total, heads, d), want) < limit
    last = [int(starts[e + 1]) - 1 for e in range(entries)]
    position1 = torch.tensor([n - 1 for n in lengths], dtype=torch.int32, device=DEV)
    for cluster in ("8", "8p", "16", "16p", "0"):
        os.environ["VIPERA_ATTENTION_CLUSTER"] = cluster
        try:
            out1 = torch.full((entries, heads * d), float("nan"), dtype=dtype, device=DEV)
            ops.attention_decode(qd[last].contiguous(), out1, kp, vp, positions=position1, block_table=tb, window=0, chunk=chunk,
                                 num_splits=splits, scratch=scratch, gate=wide_d[last].contiguous(), **common)
        finally:
            os.environ.pop("VIPERA_ATTENTION_CLUSTER", None)
        assert _rel(out1.float().cpu().view(entries, heads, d), want[last]) < limit, cluster


# heads, values per head, groups, state, norm groups; tokens of the entries of one step and whether they are fresh
SCANS = {
    "usual": ((8, 64, 2, 128, 2), [(300, 1), (128, 0), (1, 0), (2, 0), (129, 1), (1, 1), (127, 0)]),
    "one_group": ((12, 64, 1, 64, 1), [(257, 0), (3, 1), (384, 0)]),
    "small": ((3, 20, 3, 24, 5), [(77, 1), (1, 0), (140, 0), (0, 0), (16, 0)]),
    "odd": ((2, 9, 1, 19, 3), [(130, 0), (1, 0), (33, 1)]),
    "one": ((1, 1, 1, 1, 1), [(150, 0), (5, 1)]),
    "wide_values": ((4, 130, 2, 32, 4), [(200, 0), (1, 0), (64, 1)]),
    "large_state": ((2, 72, 1, 256, 2), [(140, 1), (130, 0)]),
    "single": ((6, 48, 2, 80, 3), [(1, 0), (1, 1), (1, 0)]),
    "many_entries": ((4, 16, 2, 16, 1), [(2 + i % 5 if i % 3 else 1, i % 2) for i in range(70)]),
    "one_part": ((40, 128, 4, 16, 1), [(50, 0), (1, 0)]),
}


@pytest.mark.parametrize("form", ["walk32", "walk16", "chunks"])
@pytest.mark.parametrize("name", sorted(SCANS))
def test_the_recurrence(name, form):
    """Long and short entries, fresh ones and ones that go on, single tokens beside portions, entries without
    tokens; slots in a shuffled order, of which those no entry names stay as they are.  Step sizes from tiny to
    large: states that keep everything and states that keep nothing."""
    ops = _ops()
    (heads, size, groups, n, norm_groups), described = SCANS[name]
    dtype = torch.float32 if form == "walk32" else torch.bfloat16
    counts = [c for c, _ in described]
    g = torch.Generator().manual_seed(heads * 100 + size)
    tokens, entries, inner = sum(counts), len(counts), heads * size
    xbc = torch.randn(tokens, inner + 2 * groups * n, generator=g).to(dtype)
    z_off, dt_off = 3, 3 + inner + 4
    proj = torch.randn(tokens, dt_off + heads + 2, generator=g)
    proj[:, dt_off:dt_off + heads] *= 2.0
    dt_bias, a, d = torch.linspace(-5.0, 2.0, heads), -torch.exp(torch.linspace(-3.0, 1.0, heads)), torch.randn(heads, generator=g)
    weight, eps = 1 + 0.2 * torch.randn(inner, generator=g), 1e-3
    slots = torch.randperm(entries + 3, generator=g)[:entries].to(torch.int32)
    state0 = torch.randn(entries + 3, heads * n * size, generator=g)
    fresh = torch.tensor([f for _, f in described], dtype=torch.int32)
    starts = torch.tensor(np.concatenate([[0], np.cumsum(counts)]), dtype=torch.int32)

    x = xbc[:, :inner].double().view(tokens, heads, size)
    b = xbc[:, inner:inner + groups * n].double().view(tokens, groups, n).repeat_interleave(heads // groups, dim=1)
    c = xbc[:, inner + groups * n:].double().view(tokens, groups, n).repeat_interleave(heads // groups, dim=1)
    dt = torch.nn.functional.softplus(proj[:, dt_off:dt_off + heads].double() + dt_bias.double(), threshold=1e9)
    y, want_state = torch.zeros(tokens, heads, size, dtype=F), state0.double().clone()
    for e in range(entries):
        if not counts[e]:
            continue
        s = torch.zeros(heads, n, size, dtype=F) if fresh[e] else state0[slots[e]].double().view(heads, n, size)
        for t in range(int(starts[e]), int(starts[e + 1])):
            s = torch.exp(a.double() * dt[t])[:, None, None] * s + dt[t][:, None, None] * b[t][:, :, None] * x[t][:, None, :]
            y[t] = torch.einsum("hnp,hn->hp", s, c[t]) + d.double()[:, None] * x[t]
        want_state[slots[e]] = s.reshape(-1)
    z = proj[:, z_off:z_off + inner].double()
    gated = (y.reshape(tokens, inner) * z * torch.sigmoid(z)).view(tokens, norm_groups, -1)
    want = (gated / torch.sqrt((gated * gated).mean(-1, keepdim=True) + eps)).reshape(tokens, inner) * weight.double()

    state = state0.to(DEV)
    y_d = torch.full((tokens, inner), float("nan"), device=DEV)
    out = torch.full((tokens, inner), float("nan"), dtype=dtype, device=DEV)
    jobs = ops.mamba2_jobs(tokens, entries)
    chunks = None
    if form == "chunks":
        chunks = (torch.full((jobs, heads * n * size), float("nan"), device=DEV),
                  torch.full((jobs, 2 * heads * n * size), float("nan"), dtype=torch.bfloat16, device=DEV),
                  torch.full((jobs, heads), float("nan"), device=DEV))
    ops.mamba2(xbc.to(DEV), proj.to(DEV), z_off=z_off, dt_off=dt_off, heads=heads, vdim=size, groups=groups, states=n,
               dt_bias=dt_bias.to(DEV), a=a.to(DEV), d=d.to(DEV), state=state, entry_starts=starts.to(DEV), state_slots=slots.to(DEV),
               fresh=fresh.to(DEV), num_entries=entries, any_single=1 in counts, y=y_d, norm_weight=weight.to(DEV),
               norm_groups=norm_groups, eps=eps, out=out, chunks=chunks)
    # the chunked form carries 16 bits of what it multiplies in 32-bit on the way
    limit = 1e-4 if form == "chunks" else 1e-5
    assert _rel(y_d.cpu().double(), y.reshape(tokens, inner)) < limit
    assert _rel(state.cpu().double(), want_state) < limit
    untouched = [i for i in range(entries + 3) if i not in slots.tolist()]
    assert torch.equal(state.cpu()[untouched], state0[untouched])
    assert _rel(out.float().cpu(), want) < (2e-5 if form == "walk32" else 6e-3)


@pytest.mark.parametrize("heads,groups,blocks", [(64, 8, 8), (12, 3, 4), (6, 3, 2), (5, 1, 1)])
def test_heads_that_share_their_scores(heads, groups, blocks, monkeypatch):
    """Several heads of a group to a block give what one head to a block gives."""
    ops = _ops()
    size, n, tokens = 40, 48, 200
    g = torch.Generator().manual_seed(heads)
    inner = heads * size
    args = dict(z_off=0, dt_off=inner, heads=heads, vdim=size, groups=groups, states=n, dt_bias=torch.randn(heads, generator=g).to(DEV),
                a=-torch.rand(heads, generator=g).to(DEV), d=torch.randn(heads, generator=g).to(DEV),
                entry_starts=torch.tensor([0, 150, 200], dtype=torch.int32, device=DEV),
                state_slots=torch.tensor([1, 0], dtype=torch.int32, device=DEV), fresh=torch.tensor([0, 1], dtype=torch.int32, device=DEV),
                num_entries=2, any_single=False, norm_weight=torch.ones(inner, device=DEV), norm_groups=groups, eps=1e-5)
    xbc = torch.randn(tokens, inner + 2 * groups * n, generator=g).to(torch.bfloat16).to(DEV)
    proj = torch.randn(tokens, inner + heads, generator=g).to(DEV)
    start = torch.randn(2, heads * n * size, generator=g).to(DEV)
    results = []
    for wanted in (1, blocks):
        monkeypatch.setattr(ops, "mamba2_heads_per_block", lambda *a, wanted=wanted: wanted)
        state, y = start.clone(), torch.full((tokens, inner), float("nan"), device=DEV)
        out = torch.full((tokens, inner), float("nan"), dtype=torch.bfloat16, device=DEV)
        jobs = ops.mamba2_jobs(tokens, 2)
        ops.mamba2(xbc, proj, state=state, y=y, out=out, **args,
                   chunks=(torch.empty(jobs, heads * n * size, device=DEV),
                           torch.empty(jobs, 2 * heads * n * size, dtype=torch.bfloat16, device=DEV),
                           torch.empty(jobs, heads, device=DEV)))
        results.append((state, y, out))
    assert all(torch.equal(one, other) and torch.isfinite(one.float()).all() for one, other in zip(*results))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens,hidden,ff,experts,always,top,tile_rows", [
    (3, 72, 24, 5, 2, 2, 8), (1, 100, 9, 3, 0, 3, 8), (40, 72, 24, 5, 2, 2, 32), (9, 256, 64, 8, 2, 2, 8),
    (150, 256, 64, 8, 2, 2, 128), (70, 384, 112, 30, 0, 6, 128), (33, 64, 16, 1, 1, 1, 128)])
@pytest.mark.parametrize("gated", [True, False])
def test_mixture_whose_weights_multiply_the_input(tokens, hidden, ff, experts, always, top, tile_rows, gated, dtype):
    """The experts' weights on what they read, the shared unit's on its output, in all three forms; with units
    that have no gate too."""
    ops = _ops()
    g = torch.Generator().manual_seed(tokens + hidden)
    matrices, slots = experts + always, top + always
    h = torch.randn(tokens, hidden, generator=g).to(dtype)
    router = torch.randn(experts + (1 if always else 0), hidden, generator=g) * 0.3
    gate, up = ((torch.randn(matrices, ff, hidden, generator=g) * 0.2).to(dtype) for _ in range(2))
    down = (torch.randn(matrices, hidden, ff, generator=g) * 0.2).to(dtype)
    z = h.double() @ router.double().T
    ranked = z[:, :experts].sort(dim=-1, descending=True)
    margin = ranked.values[:, top - 1] - ranked.values[:, top] if top < experts else torch.full((tokens,), float("inf"), dtype=F)
    want = torch.zeros(tokens, hidden, dtype=F)
    for t in range(tokens):
        places = [(int(e), float(torch.sigmoid(z[t, e])), 1.0) for e in ranked.indices[t, :top]]
        places += [(experts + i, 1.0, float(torch.sigmoid(z[t, experts]))) for i in range(always)]
        for e, inside, outside in places:
            x = inside * h[t].double()
            first, second = gate[e].double() @ x, up[e].double() @ x
            act = first * torch.sigmoid(first) * second if gated else torch.relu(second) ** 2
            want[t] += outside * (down[e].double() @ act)
    chosen = torch.full((tokens, slots), -7, dtype=torch.int32, device=DEV)
    weight = torch.full((tokens, slots), float("nan"), device=DEV)
    capacity = ops.moe_capacity(tokens, slots, matrices)
    group = ops.MOE_GATE_GROUP if dtype == torch.bfloat16 and ff % ops.MOE_GATE_GROUP == 0 else ff
    first = torch.stack([gate.view(matrices, ff // group, group, hidden), up.view(matrices, ff // group, group, hidden)], dim=2).reshape(
        matrices, 2 * ff, hidden) if gated else up
    expected = 32 if tile_rows == 128 and dtype == torch.float32 else tile_rows
    assert ops.moe_form(tokens, slots, hidden, ff, group if gated else ops.MOE_GATE_GROUP, dtype)[0] == expected
    rows = torch.full((tokens, slots * hidden), float("nan"), device=DEV)
    ops.moe(h.to(DEV), router=router.to(DEV), gate_up=first.contiguous().to(DEV), down=down.to(DEV), gate_group=group, top=top, groups=1,
            keep=1, group_top=1, softmax_scores=False, renormalize=False, activation=ops.ACT_SILU if gated else ops.ACT_RELU2,
            chosen=chosen, weight=weight, scratch=torch.zeros(ops.moe_scratch_words(tokens, slots, matrices), dtype=torch.int32, device=DEV),
            act=torch.full((capacity, ff), float("nan"), dtype=dtype, device=DEV), rows=rows,
            xs=torch.full((capacity, hidden), float("nan"), dtype=dtype, device=DEV), ys=torch.full((capacity, hidden), float("nan"), device=DEV),
            gated=gated, always=always, always_gate=bool(always), input_weight=True)
    ops.check_kernel_status(torch.device(DEV))
    got = rows.view(tokens, slots, hidden).double().sum(1).cpu()
    clear = margin > 1e-4
    assert torch.isfinite(got).all() and clear.float().mean() > 0.9
    assert _rel(got[clear], want[clear]) < (2e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("blocks", [("parallel", "prenorm_mixer"), ("prenorm_mixer", "parallel"), ("prenorm_mixer", "prenorm_mixer")])
def test_the_embedding_joins_again_whatever_arrangement_follows(blocks, dtype):
    """Two attention layers that run three times: whether the first of them adds what is pending itself or finds
    the stream complete, and whether the layer before it left branches, the embedding's rows join once a pass."""
    import dataclasses

    import plain_zugutar as plain
    import zugutar_cases as cases
    from vipera_rs_b200.cache import CachePools
    from vipera_rs_b200.config import architecture_of
    from vipera_rs_b200.config.spec import LayerSpec
    from vipera_rs_b200.engine.loader import build_kernels
    from vipera_rs_b200.engine.runner import ModelRunner, StepInput
    from vipera_rs_b200.parts.model import DecoderModel, model_schema
    from vipera_rs_b200.weights import RandomSource

    data = cases.config([cases.attention(), cases.attention(heads=3, kv_heads=1)], loop=(0, 2, 3))
    arch = architecture_of(data)
    spec = arch.model_spec(arch.config_from_dict(data))
    layers = [LayerSpec(block, layer.prefix, layer.parts, layer.names, {"hidden_size": spec.hidden_size, "shared_norm": True})
              for block, layer in zip(blocks, spec.layers)]
    spec = dataclasses.replace(spec, layers=layers)
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
    want = plain.forward(data, w, tokens)
    assert _rel(got, want) < (1e-5 if dtype == "float32" else 4e-2)
