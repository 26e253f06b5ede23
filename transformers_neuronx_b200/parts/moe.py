"""A feed-forward of routed experts: each token runs `top` of `n_experts` small feed-forwards (gated, or
down(relu(up x)^2) without a gate; the router may have a bias, add a correction to the scores for the choice only, restrict the choice
to the best groups of experts, scale the weights, and choose identity experts, which return their input:
parts/spec.py: RoutedFeedForwardSpec).

  z = W_router h (32-bit sums), s = sigmoid(z) or softmax(z); the `top` largest scores choose the experts
  w_j = s[e_j], or s[e_j] / sum_j s[e_j] with `renormalize`
  expert(x) = W_down (g * sigmoid(act_alpha g) * (u + up_shift)),  g = min(W_gate x, gate_limit),
              u = clamp(W_up x, -up_limit, up_limit)
  result = sum_j expert_{e_j}(w_j h)  (weight_on_input)   or   sum_j w_j expert_{e_j}(h)
           (+ gate * shared(h), a gated feed-forward that every token runs; gate = sigmoid(W_sg h), or 1)

A shared feed-forward of the experts' own form whose inner width is theirs, or a small multiple, is one or a few more
experts that every token takes with weight `gate`: it rides in the experts' products.  Any other runs as the gated
feed-forward it is, behind them; so does the former in a step of many tokens, where a dense product of its own is the faster
one.  The gate is one more row of the router's product either way.

The experts' matrices are kept stacked, [E, 2 ff, hidden] (gate rows, then up rows) and [E, hidden, ff], in the type
they are stored in.  A step routes on the device (no read on the host: the part is graph-safe) and then takes one of
two forms: in a 16-bit engine the (token, expert) pairs are sorted by expert and run as grouped products on the tensor
cores (csrc/moe_grouped.cu, csrc/gemm_tc.cu); the 32-bit engine, and sizes the tensor-core product refuses, stream the
chosen experts' matrices through the multiply-add units (csrc/moe.cu).
"""
from __future__ import annotations

import math

import torch

from ..kernels import ops
from ..weights.loader import TensorSpec
from .base import FeedForward, to_device, weight_to_device
from .linear import linear_forward
from .registry import build_part, register_feed_forward
from .spec import GatedFeedForwardSpec, RoutedFeedForwardSpec


class RoutedExperts(FeedForward):
    graph_safe = True
    can_overwrite = True

    @property
    def libraries(self):
        apart = ("gated_act", "gemm_simt") if self.folded else ()
        return ("moe", "moe_grouped", "gemm_tc") + apart + (tuple(self.shared.libraries) if self.shared is not None and not self.folded else ())

    # Rows from which the grouped tensor-core form runs in a 16-bit engine.  Measured at width 2048 (8 experts of inner
    # width 2816, 2 a token): a decode step of 1 / 8 / 32 requests takes 0.48 / 0.75 / 1.03 ms with it and 0.52 / 1.10 /
    # 2.54 ms with the kernels that stream the matrices through the multiply-add units, so it always runs.
    GROUPED_FROM = 1
    APART_FROM = 1024      # tokens from which a folded shared feed-forward runs as dense products all the same
    FOLD_MOST = 4          # a shared feed-forward of up to so many experts' widths rides in their products

    def __init__(self, spec: RoutedFeedForwardSpec):
        s = self.spec = spec
        self.n_outputs = s.n_experts + s.n_identity          # of the router
        if s.n_experts < 1 or s.n_identity < 0 or not (1 <= s.top <= self.n_outputs) or len(s.experts) != s.n_experts:
            raise ValueError(f"{s.top} of {s.n_experts} experts ({len(s.experts)} listed) and {s.n_identity} identity experts is not a choice")
        if s.top > 16 or self.n_outputs > 1024:
            raise ValueError("the routing kernel takes up to 16 chosen of up to 1024 experts")
        if s.scores not in ("sigmoid", "softmax"):
            raise ValueError(f"unknown scores {s.scores!r}: sigmoid or softmax")
        if s.expert_form not in ops.EXPERT_FORMS:
            raise ValueError(f"unknown expert form {s.expert_form!r}: {sorted(ops.EXPERT_FORMS)}")
        self.gated = s.expert_form == "gated_swish"
        if any((e.gate is None) == self.gated for e in s.experts):
            raise ValueError(f"experts of form {s.expert_form!r} {'need' if self.gated else 'have no'} gate matrices")
        if s.n_groups < 1 or self.n_outputs % s.n_groups or not (1 <= s.keep_groups <= s.n_groups) or s.group_top < 1:
            raise ValueError(f"{self.n_outputs} experts in {s.n_groups} groups of which {s.keep_groups} are kept is not a choice")
        if s.keep_groups * (self.n_outputs // s.n_groups) < s.top:
            raise ValueError(f"the {s.keep_groups} kept groups hold fewer than {s.top} experts")
        if s.shared_gate and s.shared is None:
            raise ValueError("a gate on the shared feed-forward needs one")
        self.shared = build_part("feed_forward", s.shared)
        sh = s.shared
        if sh is not None and not isinstance(sh, GatedFeedForwardSpec):
            raise ValueError("the shared feed-forward of routed experts is a gated one")
        times = sh.up.out_features // s.ff if sh is not None and sh.up.out_features % s.ff == 0 else 0
        self.folded = (1 <= times <= self.FOLD_MOST and self.gated and sh.activation == "silu"
                       and not (sh.gate.bias or sh.up.bias or sh.down.bias) and s.act_alpha == 1.0 and s.up_shift == 0.0
                       and s.gate_limit is None and s.up_limit is None and not s.weight_on_input
                       and s.top + times <= 16 and self.n_outputs + times <= 1024)
        self.always = times if self.folded else 0            # experts that every token takes
        self.router = self.gate_up = self.down = self.correction = self.router_bias = self.shared_down = None

    def tensor_specs(self):
        s = self.spec
        E = self.n_outputs
        out = [TensorSpec(s.router, (E, s.hidden), "matrix")]
        if s.correction:
            out.append(TensorSpec(s.correction, (E,), "bias"))
        if s.router_bias:
            out.append(TensorSpec(s.router_bias, (E,), "bias"))
        if s.shared_gate:
            out.append(TensorSpec(s.shared_gate, (1, s.hidden), "matrix"))
        for e in s.experts:
            if self.gated:
                out.append(TensorSpec(e.gate, (s.ff, s.hidden), "matrix"))
            out += [TensorSpec(e.up, (s.ff, s.hidden), "matrix"), TensorSpec(e.down, (s.hidden, s.ff), "matrix")]
        return out + (self.shared.tensor_specs() if self.shared is not None else [])

    def load(self, tensors, device, act_dtype):
        s = self.spec
        self.router = weight_to_device(tensors[s.router], device, act_dtype, s.router)
        if s.shared_gate:                                    # one more row of the router's product
            gate = weight_to_device(tensors[s.shared_gate], device, act_dtype, s.shared_gate)
            if gate.dtype != self.router.dtype:
                self.router, gate = self.router.float(), gate.float()
            self.router = torch.cat([self.router, gate]).contiguous()
        if s.correction:
            self.correction = to_device(tensors[s.correction], device, torch.float32)
        if s.router_bias:
            self.router_bias = to_device(tensors[s.router_bias], device, torch.float32)
        if self.shared is not None and not self.folded:
            self.shared.load(tensors, device, act_dtype)
        first = weight_to_device(tensors[s.experts[0].up], device, act_dtype, s.experts[0].up)
        # gate rows, then up rows; experts without a gate: the up rows alone
        n_mats = s.n_experts + self.always
        self.gate_up = torch.empty((n_mats, (2 if self.gated else 1) * s.ff, s.hidden), dtype=first.dtype, device=device)
        self.down = torch.empty((n_mats, s.hidden, s.ff), dtype=first.dtype, device=device)
        for i, e in enumerate(s.experts):
            mats = ((e.gate, self.gate_up[i, :s.ff]), (e.up, self.gate_up[i, s.ff:]), (e.down, self.down[i])) if self.gated \
                else ((e.up, self.gate_up[i]), (e.down, self.down[i]))
            for name, dst in mats:
                w = weight_to_device(tensors[name], device, act_dtype, name)
                if w.dtype != first.dtype:
                    raise ValueError(f"{name} is stored as {w.dtype}, the other experts' matrices as {first.dtype}")
                dst.copy_(w)
        if self.folded:                                      # slices of the shared feed-forward's inner width
            sh = s.shared
            whole = [weight_to_device(tensors[l.weight], device, act_dtype, l.weight) for l in (sh.gate, sh.up, sh.down)]
            for w, l in zip(whole, (sh.gate, sh.up, sh.down)):
                if w.dtype != first.dtype:
                    raise ValueError(f"{l.weight} is stored as {w.dtype}, the experts' matrices as {first.dtype}")
            for j in range(self.always):
                i, part = s.n_experts + j, slice(j * s.ff, (j + 1) * s.ff)
                self.gate_up[i, :s.ff].copy_(whole[0][part])
                self.gate_up[i, s.ff:].copy_(whole[1][part])
                self.down[i].copy_(whole[2][:, part])
            if act_dtype != torch.float32:
                self.shared_down = whole[2]                  # for steps of many tokens; the other two lie in gate_up as they are

    def parameter_bytes(self):
        return sum(t.numel() * t.element_size() for t in (self.router, self.gate_up, self.down, self.correction, self.router_bias)
                   if t is not None) + (self.shared.parameter_bytes() if self.shared is not None and not self.folded else 0)

    def step_bytes(self, n_tokens: int) -> int:
        """Bytes of weights a step of n_tokens is expected to read: every expert once that some token chooses, with
        tokens that choose independently and evenly."""
        s = self.spec
        used = s.n_experts * (1.0 - (1.0 - s.top / self.n_outputs) ** n_tokens)
        per = (self.gate_up[0].numel() + self.down[0].numel()) * self.gate_up.element_size()
        shared = 0 if self.shared is None else (per * self.always if self.folded else self.shared.parameter_bytes())
        return int(self.router.numel() * self.router.element_size() + used * per) + shared

    def forward(self, ctx, h, out, accumulate=True):
        s, N = self.spec, h.shape[0]
        apart = self.shared_down is not None and N >= self.APART_FROM and ops.moe_grouped_supported(h, self.gate_up, self.down)
        always = 0 if apart else self.always
        gate = ctx.scratch(1, N, torch.float32).view(-1) if s.shared_gate and always == 0 else None
        ids = ctx.scratch(N, s.top + always, torch.int32)
        weights = ctx.scratch(N, s.top + always, torch.float32)
        ops.moe_route(h, self.router, ctx.token_request, ids, weights, s.top, softmax_scores=s.scores == "softmax",
                      renormalize=s.renormalize, correction=self.correction, n_groups=s.n_groups, keep_groups=s.keep_groups,
                      group_top=s.group_top, renorm_eps=s.renorm_eps, weight_scale=s.weight_scale, bias=self.router_bias, always=always,
                      n_identity=s.n_identity, gated=bool(s.shared_gate), gate_out=gate)
        inf = math.inf
        limits = (s.gate_limit if s.gate_limit is not None else inf, -s.up_limit if s.up_limit is not None else -inf,
                  s.up_limit if s.up_limit is not None else inf)
        if N >= self.GROUPED_FROM and ops.moe_grouped_supported(h, self.gate_up, self.down):
            E = s.n_experts + always
            ops.moe_grouped(ctx, h, self.gate_up[:E], self.down[:E], ids, weights, out, *limits, s.act_alpha, s.up_shift,
                            weight_on_input=s.weight_on_input, accumulate=accumulate, form=s.expert_form)
        else:
            pairs = N * (s.top + always)
            y = ctx.scratch(pairs, s.ff)
            ops.moe_experts(h, self.gate_up, self.down, ids, weights, y, out, *limits, s.act_alpha, s.up_shift,
                            weight_on_input=s.weight_on_input, accumulate=accumulate,
                            per_pair=ctx.scratch(pairs, s.hidden, torch.float32), form=s.expert_form)
        if apart:
            self._shared_apart(ctx, h, out, gate)
        elif self.shared is not None and not self.folded:
            if gate is None:
                self.shared.forward(ctx, h, out)
            else:
                self.shared.forward(ctx, h, out, row_scale=gate)

    def _shared_apart(self, ctx, h, out, gate):
        """The folded shared feed-forward as dense products: its slices' gate and up rows are neighbours in gate_up, so a token's
        output is `always` rows [gate | up] of the activation kernel, whose results lie in the order of the inner width."""
        s, N, n = self.spec, h.shape[0], self.always
        gu, a = ctx.scratch(N, n * 2 * s.ff), ctx.scratch(N, n * s.ff)
        linear_forward(h, self.gate_up[s.n_experts:].view(n * 2 * s.ff, s.hidden), None, gu)
        ops.gated_activation(gu.view(N * n, 2 * s.ff), a.view(N * n, s.ff), "silu", gate)
        linear_forward(a, self.shared_down, None, out, residual=out)


register_feed_forward("routed_experts", RoutedExperts)
