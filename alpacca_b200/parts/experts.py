"""A feed-forward of routed experts with a grouped router.

    z = W_r h (32-bit);  s = softmax(z) over all experts
    the experts form `groups` equal groups of neighbours; a group's score is its largest s; only experts of the
    `keep` best groups can be chosen; the `top` largest s among them are chosen
    weights = chosen s / (their sum + 1e-20) * scale;  output = sum of weight * expert(h)
    expert(h) = W_down act(W_up h), no biases

Options: `router_bias` (a bias on the logits, tensor `<router>.b`); `gate_name`: gated experts,
expert(h) = W_down (act(W_gate h) * (W_up h)).  With one group, all of it kept and scale 1 the weights are the
softmax over the chosen logits alone (exp(z_j) / sum over the chosen of exp(z)), which is the router of designs that
choose by logit.

`score` "sigmoid" (or "logit"): s = sigmoid(z) (or z) instead of the softmax; `correction` names a tensor [experts]
that is added to s for the CHOICE alone (groups and experts are chosen by s + correction, the weights are the chosen
s); `group_top`: a group's score is the sum of that many of its largest choice scores; `renorm` off: the weights are
not divided by their sum.

The experts' matrices are stacked ([experts, ff, width] and, side by side, [width, experts, ff]) so that a
kernel picks an expert by index from device memory: routing never reaches the host, and a step with routed
experts is captured in a CUDA graph like any other (csrc/moe.cu).  Steps of few tokens read the chosen
experts' rows per (token, expert) pair; steps of many tokens run all experts in two library products with the
weights of experts that were not chosen set to zero (`ops.moe_experts`).
"""
from __future__ import annotations

import torch

from .. import ops
from ..weights.loader import ParamSpec, WeightError
from .base import BuildOptions, FeedForward


class RoutedExperts(FeedForward):
    def __init__(self, opts: BuildOptions, width: int, inner: int, n_experts: int, top: int, groups: int, keep: int,
                 scale: float, prefix: str, activation: str = "gelu", router_name: str = "router",
                 expert_names=("e{}.up", "e{}.down"), router_bias: bool = False, gate_name: str | None = None,
                 score: str = "softmax", correction: str | None = None, group_top: int = 1, renorm: bool = True):
        if activation not in ops.MOE_ACTIVATIONS:
            raise ValueError(f"activation must be one of {tuple(ops.MOE_ACTIVATIONS)}, got {activation!r}")
        if n_experts % groups or not 0 < keep <= groups or not 0 < top <= keep * (n_experts // groups):
            raise ValueError(f"{n_experts} experts in {groups} groups, {keep} kept, {top} chosen cannot be routed")
        self.opts, self.width, self.inner, self.E = opts, int(width), int(inner), int(n_experts)
        self.top, self.groups, self.keep, self.scale = int(top), int(groups), int(keep), float(scale)
        self.prefix, self.activation, self.router_name, self.expert_names = prefix, activation, router_name, expert_names
        self.router_bias, self.gate_name = bool(router_bias), gate_name
        if score not in ops.MOE_SCORES or (score == "softmax" and (correction or group_top != 1 or not renorm)):
            raise ValueError(f"{prefix}: score {score!r} with correction {correction!r}, group_top {group_top}, renorm "
                             f"{renorm} is not a router of this part")
        self.score, self.correction_name, self.group_top, self.renorm = score, correction, int(group_top), bool(renorm)
        self.correction = None
        self.router = self.bias = self.w_up = self.w_down = self.w_gate_up = None

    def own_param_specs(self):
        up, down = self.expert_names
        specs = [ParamSpec(f"{self.prefix}.{self.router_name}", (self.E, self.width), "vector", "normal")]
        for e in range(self.E):
            specs.append(ParamSpec(f"{self.prefix}.{up.format(e)}", (self.inner, self.width), "matrix", "normal"))
            specs.append(ParamSpec(f"{self.prefix}.{down.format(e)}", (self.width, self.inner), "matrix", "normal"))
        if self.gate_name is not None:
            specs += [ParamSpec(f"{self.prefix}.{self.gate_name.format(e)}", (self.inner, self.width), "matrix", "normal")
                      for e in range(self.E)]
        if self.router_bias:
            specs.append(ParamSpec(f"{self.prefix}.{self.router_name}.b", (self.E,), "vector", "normal"))
        if self.correction_name is not None:
            specs.append(ParamSpec(f"{self.prefix}.{self.correction_name}", (self.E,), "vector", "normal"))
        return specs

    def load_own(self, fetch):
        specs = self.own_param_specs()
        self.router = fetch(specs[0])
        ups = [fetch(s) for s in specs[1:1 + 2 * self.E:2]]
        self.w_down = torch.stack([fetch(s) for s in specs[2:2 + 2 * self.E:2]], dim=1).contiguous()      # [width, E, ff]
        if self.gate_name is not None:
            gates = [fetch(s) for s in specs[1 + 2 * self.E:1 + 3 * self.E]]
            self.w_gate_up = torch.stack([torch.stack(gates), torch.stack(ups)]).contiguous()      # [2, E, ff, width]
            self.w_up = self.w_gate_up[1]
        else:
            self.w_up = torch.stack(ups).contiguous()
        if self.router_bias:
            self.bias = fetch(specs[1 + (3 if self.gate_name is not None else 2) * self.E])
        if self.correction_name is not None:
            self.correction = fetch(specs[-1])

    def forward(self, h, ctx):
        T = ctx.n_tokens
        idx, wts = ops.moe_route(h, self.router, T, self.groups, self.keep, self.top, self.scale, bias=self.bias,
                                 score=self.score, correction=self.correction, group_top=self.group_top,
                                 renorm=self.renorm)
        out = torch.empty((h.shape[0], self.width), dtype=h.dtype, device=h.device)
        return ops.moe_experts(h, self.w_up, self.w_down, idx, wts, out, T, self.activation, gate_up=self.w_gate_up)


class TableExperts(FeedForward):
    """Gated experts that the token's id chooses: row token of a table [vocab, top] names a token's experts (all different),
    each with weight 1 / top; there is no router.  The output is float32.

        out = sum_k E_(e_k)(h) / top + sigmoid(w_s . h) S(h),       E(h) = W_down (act(W_gate h) * (W_up h))

    `shared_inner` > 0: the shared expert S, of that inner size, runs for every token; its gate is one number per token,
    formed in 32-bit.  A block whose kernel has the stream's row in registers may form it there: `row_gate()` is the
    vector w_s, and `forward` takes the products as `gate_logits`.

    The experts' matrices are stacked, gates and up-projections interleaved in groups of 8 rows, the inner sizes padded with
    zero units to multiples of 8.  Few tokens run two skinny products that read the chosen experts' weights once
    (csrc/moe_gemv.cu); many tokens grouped products over the (token, expert) pairs in order of their experts (csrc/moe.cu,
    csrc/gemm_tc.cu).  The table is read by the kernels: routing never reaches the host."""

    def __init__(self, opts: BuildOptions, width: int, inner: int, n_experts: int, top: int, vocab: int, prefix: str,
                 activation: str = "silu", shared_inner: int = 0, table_name: str = "table",
                 expert_names=("e{}.gate", "e{}.up", "e{}.down"), shared_names=("shared.gate", "shared.up", "shared.down"),
                 shared_gate: str = "shared.sg"):
        if activation not in ops.MOE_ACTIVATIONS:
            raise ValueError(f"activation must be one of {tuple(ops.MOE_ACTIVATIONS)}, got {activation!r}")
        if not 0 < top <= n_experts:
            raise ValueError(f"{prefix}: {top} of {n_experts} experts cannot be chosen")
        self.opts, self.width, self.inner, self.E, self.top = opts, int(width), int(inner), int(n_experts), int(top)
        self.vocab, self.prefix, self.activation, self.shared_inner = int(vocab), prefix, activation, int(shared_inner)
        self.table_name, self.expert_names, self.shared_names, self.shared_gate = table_name, expert_names, shared_names, shared_gate
        self.table = self.gate_up = self.down = self.shared_gate_up = self.shared_down = self.w_sg = None

    def own_param_specs(self):
        p = self.prefix
        specs = [ParamSpec(f"{p}.{self.table_name}", (self.vocab, self.top), "int", f"choice:{self.E}")]
        gate, up, down = self.expert_names
        for e in range(self.E):
            specs += [ParamSpec(f"{p}.{gate.format(e)}", (self.inner, self.width)),
                      ParamSpec(f"{p}.{up.format(e)}", (self.inner, self.width)),
                      ParamSpec(f"{p}.{down.format(e)}", (self.width, self.inner))]
        if self.shared_inner:
            gate, up, down = self.shared_names
            specs += [ParamSpec(f"{p}.{gate}", (self.shared_inner, self.width)),
                      ParamSpec(f"{p}.{up}", (self.shared_inner, self.width)),
                      ParamSpec(f"{p}.{down}", (self.width, self.shared_inner)),
                      ParamSpec(f"{p}.{self.shared_gate}", (1, self.width), "vector")]
        return specs

    def load_own(self, fetch):
        specs = self.own_param_specs()
        self.table = fetch(specs[0])
        if int(self.table.min()) < 0 or int(self.table.max()) >= self.E:
            raise WeightError(f"{specs[0].name} names experts outside 0..{self.E - 1}")
        ff = -(-self.inner // 8) * 8
        for e in range(self.E):
            gate_up, down = self._laid_out(*(fetch(s) for s in specs[1 + 3 * e:4 + 3 * e]))
            if e == 0:
                self.gate_up = torch.empty((self.E, 2 * ff, self.width), dtype=down.dtype, device=down.device)
                self.down = torch.empty((self.E, self.width, ff), dtype=down.dtype, device=down.device)
            self.gate_up[e], self.down[e] = gate_up, down
        self.gate_up, self.down = self.gate_up.view(-1, self.width), self.down.view(-1, ff)
        if self.shared_inner:
            self.shared_gate_up, self.shared_down = self._laid_out(*(fetch(s) for s in specs[1 + 3 * self.E:4 + 3 * self.E]))
        if self.shared_inner:
            self.w_sg = fetch(specs[-1]).reshape(-1).contiguous()

    def _laid_out(self, gate, up, down):
        """(gate|up in groups of 16 rows: the gates of 8 units, then their up-projections; down), padded to whole groups."""
        more = -gate.shape[0] % 8
        gate, up = (torch.nn.functional.pad(w, (0, 0, 0, more)).view(-1, 8, self.width) for w in (gate, up))
        return (torch.cat([gate, up], dim=1).reshape(-1, self.width).contiguous(),
                torch.nn.functional.pad(down, (0, more)).contiguous())

    def shared_weights(self):
        """(gate|up, down) of the shared expert as the kernels read them, or None."""
        return (self.shared_gate_up, self.shared_down) if self.shared_inner else None

    def row_gate(self):
        """The vector (float32 [width]) whose product with this part's input is the shared expert's gate logit."""
        return self.w_sg

    def forward(self, h, ctx, gate_logits=None):
        if self.shared_inner and gate_logits is None:
            gate_logits = ops.row_dots(h, self.w_sg, ctx.n_tokens)
        out = torch.empty((h.shape[0], self.width), dtype=torch.float32, device=h.device)
        return ops.moe_shared_experts(h, self.gate_up, self.down, self.E, self.top, out, ctx, activation=self.activation,
                                      table=self.table, shared=self.shared_weights(), gate_logits=gate_logits)


class ScoredExperts(FeedForward):
    """Experts chosen by a router's scores, beside an optional shared expert that runs for every token.  The output is float32.

        z = W_r h (32-bit);  s = score(z);  the `top` largest s are chosen, their weights are s as they are
        (`renorm`: divided by their sum)
        out = sum_k E_(e_k)(s_k h) + S(h)             `weight_in`: the weight multiplies the expert's input
        out = sum_k s_k E_(e_k)(h) + S(h)             otherwise
        E(h) = W_down act(W_up h), or with gates (`expert_names` of three) W_down (act(W_gate h) * (W_up h))

    The experts' matrices are stacked, inner sizes padded with zero units to multiples of 16 (act(0) = 0); gates and
    up-projections are interleaved in groups of 8 rows.  The kernels are those of `TableExperts`."""

    def __init__(self, opts: BuildOptions, width: int, inner: int, n_experts: int, top: int, prefix: str, activation: str = "relu2",
                 score: str = "sigmoid", renorm: bool = False, weight_in: bool = False, shared_inner: int = 0,
                 router_name: str = "router", expert_names=("e{}.up", "e{}.down"), shared_names=("shared.up", "shared.down")):
        if activation not in ops.MOE_ACTIVATIONS:
            raise ValueError(f"activation must be one of {tuple(ops.MOE_ACTIVATIONS)}, got {activation!r}")
        if score not in ("sigmoid", "logit"):
            raise ValueError(f"{prefix}: score {score!r} is not one of this part's")
        if not 0 < top <= n_experts:
            raise ValueError(f"{prefix}: {top} of {n_experts} experts cannot be chosen")
        if len(expert_names) != len(shared_names) or len(expert_names) not in (2, 3):
            raise ValueError(f"{prefix}: experts have two matrices, or three with a gate, and the shared one likewise")
        self.opts, self.width, self.inner, self.E, self.top = opts, int(width), int(inner), int(n_experts), int(top)
        self.prefix, self.activation, self.score, self.renorm = prefix, activation, score, bool(renorm)
        self.weight_in, self.shared_inner, self.gated = bool(weight_in), int(shared_inner), len(expert_names) == 3
        self.router_name, self.expert_names, self.shared_names = router_name, expert_names, shared_names
        self.router = self.router16 = self.up = self.down = self.shared_up = self.shared_down = None

    def _specs_of(self, names, inner):
        shapes = [(inner, self.width)] * (len(names) - 1) + [(self.width, inner)]
        return [ParamSpec(f"{self.prefix}.{n}", s) for n, s in zip(names, shapes)]

    def own_param_specs(self):
        specs = [ParamSpec(f"{self.prefix}.{self.router_name}", (self.E, self.width), "vector", "normal")]
        for e in range(self.E):
            specs += self._specs_of([n.format(e) for n in self.expert_names], self.inner)
        if self.shared_inner:
            specs += self._specs_of(self.shared_names, self.shared_inner)
        return specs

    def load_own(self, fetch):
        specs, n = self.own_param_specs(), len(self.expert_names)
        self.router = fetch(specs[0])
        w16 = self.router.to(torch.bfloat16)
        self.router16 = w16.contiguous() if self.opts.dtype == torch.bfloat16 and torch.equal(w16.float(), self.router) else None
        ff = -(-self.inner // 16) * 16
        for e in range(self.E):
            up, down = self._laid_out(*(fetch(s) for s in specs[1 + n * e:1 + n * (e + 1)]))
            if e == 0:
                self.up = torch.empty((self.E, *up.shape), dtype=up.dtype, device=up.device)
                self.down = torch.empty((self.E, *down.shape), dtype=down.dtype, device=down.device)
            self.up[e], self.down[e] = up, down
        self.up, self.down = self.up.view(-1, self.width), self.down.view(-1, ff)
        if self.shared_inner:
            self.shared_up, self.shared_down = self._laid_out(*(fetch(s) for s in specs[1 + n * self.E:]))

    def _laid_out(self, *matrices):
        """(gate|up in groups of 16 rows, or up; down), the inner size padded to a multiple of 16."""
        *first, down = matrices
        more = -down.shape[1] % 16
        first = [torch.nn.functional.pad(w, (0, 0, 0, more)) for w in first]
        if self.gated:
            first = [torch.cat([w.view(-1, 8, self.width) for w in first], dim=1).reshape(-1, self.width)]
        return first[0].contiguous(), torch.nn.functional.pad(down, (0, more)).contiguous()

    def forward(self, h, ctx):
        choice = ops.moe_route(h, self.router, ctx.n_tokens, 1, 1, self.top, 1.0, score=self.score, renorm=self.renorm,
                               router16=self.router16)
        out = torch.empty((h.shape[0], self.width), dtype=torch.float32, device=h.device)
        shared = (self.shared_up, self.shared_down) if self.shared_inner else None
        return ops.moe_shared_experts(h, self.up, self.down, self.E, self.top, out, ctx, activation=self.activation,
                                      choice=choice, shared=shared, gated=self.gated, weight_in=self.weight_in)
