"""Mamba-2's recurrence (state-space duality) as a mixer with a state of fixed size.

From the mixer's input h: ``[z | x | B | C | dt] = W_in h`` (``inner = num_heads * value_dim`` values of z and
of x, ``groups * state`` of B and of C, one dt per head); x, B and C together pass a causal convolution per
channel (with bias) and silu; ``dt = softplus(dt + dt_bias)``.  Per head, whose B and C are those of group
``head // (num_heads / groups)``, a matrix S [state, value_dim] in 32-bit floats, zero at a request's start:

    S = exp(-exp(A_log) dt) S + dt B x^T        y = S^T C + D x

The concatenated y is multiplied by silu(z), divided by its root mean square in ``norm_groups`` equal parts,
multiplied by a weight per value and sent through the output matrix.  A request keeps S and the convolution's
last inputs.  The products run in the run's type; z, dt and the convolution's inputs stay 32-bit behind the
product, the convolution's outputs are in the run's type, and the recurrence is 32-bit
(``csrc/kernels/mamba2.cu``).
"""
from __future__ import annotations

import os

import torch

from ..config.registry import MIXERS
from ..errors import UnsupportedError
from ..kernels import ops
from ..weights import TensorSpec
from .base import CacheBundle, FixedState, Mixer
from .conv import CausalConv
from .linear import Linear


class Mamba2(Mixer):
    """params: hidden_size, num_heads, value_dim, state, groups, taps (of the convolution), norm_groups,
    norm_eps and, optionally, ``rows_name`` (the buffer of the rows it leaves where it is handed no stream).
    Tensors under ``<prefix>``: in [2 inner + 2 groups * state + heads, hidden], conv [inner + 2 groups *
    state, taps] (+ bias), dt_bias, A_log, D [heads], norm [inner], o [hidden, inner]."""

    kernels = ("mamba2", "seqconv")
    leaves_rows = True
    # Steps of this many tokens and more run their portions as chunks side by side in bfloat16; shorter
    # ones walk each entry's tokens in one launch.
    CHUNKED_FROM = int(os.environ.get("VIPERA_SSD_CHUNKED_FROM", 48))

    @staticmethod
    def _sizes(params):
        inner = int(params["num_heads"]) * int(params["value_dim"])
        return inner, inner + 2 * int(params["groups"]) * int(params["state"])

    @classmethod
    def schema(cls, params, prefix):
        hidden, heads = params["hidden_size"], params["num_heads"]
        inner, channels = cls._sizes(params)
        schema = {
            f"{prefix}.in.weight": TensorSpec((inner + channels + heads, hidden)),
            f"{prefix}.dt_bias.weight": TensorSpec((heads,), init="bias", store="float32"),
            f"{prefix}.A_log.weight": TensorSpec((heads,), init="log_rate", store="float32"),
            f"{prefix}.D.weight": TensorSpec((heads,), init="norm", store="float32"),
            f"{prefix}.norm.weight": TensorSpec((inner,), init="norm", store="float32"),
            f"{prefix}.o.weight": TensorSpec((hidden, inner)),
        }
        schema.update(CausalConv.schema(f"{prefix}.conv", channels, int(params["taps"]), bias=True))
        return schema

    def __init__(self, params, prefix, tensors, dtype, device):
        super().__init__(params, prefix, tensors, dtype, device)
        self.hidden, self.heads, self.vdim = (int(params[k]) for k in ("hidden_size", "num_heads", "value_dim"))
        self.state, self.groups, self.norm_groups = (int(params[k]) for k in ("state", "groups", "norm_groups"))
        self.norm_eps = float(params["norm_eps"])
        self.rows_name = str(params.get("rows_name", "mamba2.rows"))
        self.inner, self.channels = self._sizes(params)
        if self.heads % self.groups or self.inner % self.norm_groups:
            raise UnsupportedError(f"{prefix}: {self.groups} groups must divide {self.heads} heads, and {self.norm_groups} "
                                   f"norm groups {self.inner} values")
        if self.state > ops.MAMBA2_MAX_STATE:
            raise UnsupportedError(f"{prefix}: a state of {self.state} rows; the kernels take up to {ops.MAMBA2_MAX_STATE}")

        def kept(name):
            return tensors[f"{prefix}.{name}.weight"].to(device=device, dtype=torch.float32).contiguous()

        self.proj = Linear(tensors[f"{prefix}.in.weight"], dtype, device)
        self.out = Linear(tensors[f"{prefix}.o.weight"], dtype, device)
        self.conv = CausalConv(f"{prefix}.conv", tensors, device, add_input=False, activation="silu")
        self.dt_bias, self.d, self.norm_weight = kept("dt_bias"), kept("D"), kept("norm")
        self.a = (-torch.exp(kept("A_log"))).contiguous()

    def kernel_families(self):
        return tuple(dict.fromkeys(self.kernels + self.proj.kernel_families() + self.out.kernel_families()))

    @classmethod
    def cache_request_for(cls, params):
        _, channels = cls._sizes(params)
        size = int(params["num_heads"]) * int(params["state"]) * int(params["value_dim"])
        return CacheBundle.of(conv=CausalConv.state_request(channels, int(params["taps"])),
                              scan=FixedState((size,), torch.float32))

    @classmethod
    def workspace_bytes(cls, params, tokens, element_bytes):
        inner, channels = cls._sizes(params)
        heads = int(params["num_heads"])
        jobs = ops.mamba2_jobs(tokens, 1)
        return (tokens * ((inner + channels + heads) * 4 + channels * element_bytes + inner * (4 + element_bytes)
                          + int(params["hidden_size"]) * 4)
                + jobs * heads * (2 * int(params["state"]) * int(params["value_dim"]) + 1) * 4)

    def forward(self, ctx, h, residual, cache, writes_cache):
        count, ws = ctx.num_tokens, ctx.workspace
        proj = ws.get("mamba2.proj", (count, self.proj.out_features), torch.float32)
        self.proj(ctx, h, epilogue=ops.EPI_STORE, out=proj)
        xbc = ws.get("mamba2.xbc", (count, self.channels), ctx.dtype)
        self.conv(ctx, proj[:, self.inner:], cache.get("conv"), **({"out_f32": xbc} if ctx.dtype == torch.float32 else {"out": xbc}))
        y = ws.get("mamba2.y", (count, self.inner), torch.float32)
        mixed = ws.get("mamba2.out", (count, self.inner), ctx.dtype)
        chunks = None
        if ctx.dtype == torch.bfloat16 and not ctx.all_single and count >= self.CHUNKED_FROM:
            jobs = ops.mamba2_jobs(count, ctx.num_entries)
            chunks = (ws.get("mamba2.chunk_state", (jobs, self.heads * self.state * self.vdim), torch.float32),
                      ws.get("mamba2.chunk_start", (jobs, 2 * self.heads * self.state * self.vdim), torch.bfloat16),
                      ws.get("mamba2.chunk_decay", (jobs, self.heads), torch.float32))
        ops.mamba2(xbc, proj, z_off=0, dt_off=self.inner + self.channels, heads=self.heads, vdim=self.vdim,
                   groups=self.groups, states=self.state, dt_bias=self.dt_bias, a=self.a, d=self.d,
                   state=cache["scan"].data, entry_starts=ctx.entry_starts, state_slots=ctx.state_slots, fresh=ctx.fresh,
                   num_entries=ctx.num_entries, any_single=ctx.any_single, y=y, norm_weight=self.norm_weight,
                   norm_groups=self.norm_groups, eps=self.norm_eps, out=mixed, chunks=chunks)
        if residual is None:
            rows = ws.get(self.rows_name, (count, self.hidden), torch.float32)
            self.out(ctx, mixed, epilogue=ops.EPI_STORE, out=rows)
            return rows, 1
        self.out(ctx, mixed, epilogue=ops.EPI_RESIDUAL, resid=residual)
        return None


MIXERS.register("mamba2", Mamba2)
