"""A state-space mixer with one decay and one step size per head and token (Dao and Gu, "Transformers are SSMs: Generalized
Models and Efficient Algorithms Through Structured State Space Duality"):

    z, x (H x V each), B, C (G x N each), dt (H) = W_in h
    x, B, C   pass a short causal convolution per channel over time, with a bias, and SiLU
    dt        softplus(dt + dt_bias);   a = exp(-exp(A_log) dt)               per head; head h reads group h // (H / G)
    S         <- a S + dt B x^T    [N, V];    y = S^T C + D_h x
    out       = W_o (n(y * silu(z)) * w),  n divides each of `norm_groups` equal parts by its own root mean square

S is float32 and carried from step to step, and so are the convolution's last taps - 1 inputs: two states per sequence.
The projection leaves its product in float32, everything after it up to W_o is 32-bit arithmetic (csrc/state_space.cu), but
for prompts in bfloat16, where the convolution's outputs are rounded to bfloat16 for the tensor cores.
"""
from __future__ import annotations

import torch

from .. import ops
from ..weights.loader import ParamSpec
from .base import BuildOptions, Mixer, StateSpec
from .linear import Linear


class StateSpaceMixer(Mixer):
    def __init__(self, opts: BuildOptions, width: int, n_heads: int, vdim: int, state: int, n_groups: int, taps: int,
                 norm_groups: int, eps: float, prefix: str, names=("in", "conv", "dt_bias", "A_log", "D", "norm", "o"),
                 weight_suffix: str = "", bias_suffix: str = ".b", out_dtype=None):
        self.opts, self.prefix, self.names, self.bias_suffix = opts, prefix, names, bias_suffix
        self.width, self.H, self.V, self.N, self.G = int(width), int(n_heads), int(vdim), int(state), int(n_groups)
        self.taps, self.norm_groups, self.eps = int(taps), int(norm_groups), float(eps)
        self.inner = self.H * self.V
        self.channels = self.inner + 2 * self.G * self.N
        if self.H % self.G:
            raise ValueError(f"{prefix}: {self.H} heads cannot share {self.G} groups")
        if self.inner % self.norm_groups:
            raise ValueError(f"{prefix}: {self.inner} columns cannot be normed in {self.norm_groups} equal parts")
        if not 0 < self.N <= ops.RECURRENCE_MAX_DIM:
            raise ValueError(f"{prefix}: a state of {self.N} is outside 1..{ops.RECURRENCE_MAX_DIM}")
        if not 1 <= self.taps <= ops.SSM_MAX_TAPS:
            raise ValueError(f"{prefix}: a convolution over {self.taps} tokens is outside 1..{ops.SSM_MAX_TAPS}")
        # rows padded with zeros to whole groups of four numbers, which the kernels read 16 bytes at a time
        self.proj = Linear(opts, width, [(f"{prefix}.{names[0]}", self.inner + self.channels + self.H)],
                           out_dtype=torch.float32, weight_suffix=weight_suffix, pad_rows_to=8)
        self.out = Linear(opts, self.inner, [(f"{prefix}.{names[6]}", width)], weight_suffix=weight_suffix, out_dtype=out_dtype)
        self.conv = self.conv_bias = self.dt_bias = self.A_log = self.skip = self.norm_weight = None

    def own_param_specs(self):
        p, (_, conv, dt_bias, A_log, D, norm, _) = self.prefix, self.names
        return [ParamSpec(f"{p}.{conv}", (self.channels, self.taps), "vector", "normal"),
                ParamSpec(f"{p}.{conv}{self.bias_suffix}", (self.channels,), "vector", "normal"),
                ParamSpec(f"{p}.{dt_bias}", (self.H,), "vector", "normal"),
                ParamSpec(f"{p}.{A_log}", (self.H,), "vector", "normal"),
                ParamSpec(f"{p}.{D}", (self.H,), "vector", "one_plus_normal"),
                ParamSpec(f"{p}.{norm}", (self.inner,), "vector", "one_plus_normal")]

    def load_own(self, fetch):
        conv, self.conv_bias, self.dt_bias, self.A_log, self.skip, self.norm_weight = (fetch(s) for s in self.own_param_specs())
        self.conv = conv.t().contiguous()              # [taps, channels]: what the kernels read

    def cache_specs(self) -> list:
        """The matrix per head, and the convolution's last inputs."""
        kept = [StateSpec((self.taps - 1, self.channels), torch.float32)] if self.taps > 1 else []
        return [StateSpec((self.H, self.N, self.V), torch.float32)] + kept

    def cache_spec(self):
        specs = self.cache_specs()
        if len(specs) > 1:
            raise ValueError(f"{self.prefix}: the mixer keeps two states; the block asks `cache_specs()`")
        return specs[0]

    def _in_chunks(self, ctx) -> bool:
        return (self.opts.dtype == torch.bfloat16 and ctx.n_tokens >= ops.SSM_CHUNKS_FROM * ctx.n_seqs
                and ops.ssm_chunks_supports(self.N, self.V, self.H, self.G))

    def forward(self, h, ctx, cache, write_cache: bool = True):
        T, H, G, N, V = ctx.n_tokens, self.H, self.G, self.N, self.V
        memory, held = cache if isinstance(cache, (list, tuple)) else (cache, None)
        memory, held = memory.state, held.state if held is not None else None
        proj = self.proj.forward(h, n_rows=T)
        rows, dev = proj.shape[0], proj.device
        y = torch.empty((rows, self.inner), dtype=torch.float32, device=dev)
        in_step = ctx.is_decode and ops.ssm_step_supports(N, V)
        if in_step:
            ops.ssm_step(proj, self.conv, self.conv_bias, held, self.A_log, self.dt_bias, self.skip, memory, y, ctx, H, G, N, V,
                         write_state=write_cache)
        else:
            chunks = self._in_chunks(ctx)
            xbc = torch.empty((rows, self.channels), dtype=torch.bfloat16 if chunks else torch.float32, device=dev)
            decay = torch.empty((rows, H), dtype=torch.float32, device=dev)
            dt = torch.empty((rows, H), dtype=torch.float32, device=dev)
            ops.ssm_prepare(proj, self.conv, self.conv_bias, held, self.A_log, self.dt_bias, xbc, decay, dt, ctx, H, G, N, V,
                            log_decay=chunks, write_state=write_cache)
            if chunks:
                ops.ssm_chunks(xbc, decay, dt, self.skip, memory, y, ctx, H, G, N, V, write_state=write_cache)
            else:
                x, B, C = xbc[:, :self.inner], xbc[:, self.inner:self.inner + G * N], xbc[:, self.inner + G * N:]
                ops.gated_recurrence("scalar", C, B, x, memory, y, ctx, H, G, N, V, decay=decay, beta=dt, skip=self.skip,
                                     write_state=write_cache)
        mixed = torch.empty((rows, self.inner), dtype=self.opts.dtype, device=dev)
        ops.ssm_gate_norm(y, proj, self.norm_weight, self.norm_groups, self.eps, mixed, ctx, H, G, N, V, self.taps,
                          conv_state=held if in_step and write_cache else None)
        return self.out.forward(mixed, n_rows=T)
