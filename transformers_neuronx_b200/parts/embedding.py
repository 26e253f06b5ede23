"""The two ends of the decoder: token embedding (with the optional projection to the hidden width
and the position encoding that is added there), and the head (final norm, optional projection
back, output matrix tied to the embedding table) on the rows whose logits are wanted.

Reference: host embedding src/transformers_neuronx/opt/model.py:162-166; head
src/transformers_neuronx/layers/transformer.py:148-213 (slice the wanted column, LayerNorm,
product with lm_head, no bias; logits leave in 32-bit, base.py:641-647).
"""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorSpec
from .base import Part, to_device, weight_to_device
from .linear import Linear, linear_forward
from .registry import build_part
from .spec import EmbeddingSpec, HeadSpec, StreamJoinSpec


class Embedding(Part):
    graph_safe = True
    def __init__(self, spec: EmbeddingSpec):
        self.spec = spec
        self.table = None
        self.project_in = Linear(spec.project_in) if spec.project_in else None
        self.position = build_part("position", spec.position) if spec.position else None

    @property
    def libraries(self):
        libs = ["embedding"]
        if self.project_in is not None:
            libs += list(self.project_in.libraries)
        if self.position is not None:
            libs += list(self.position.libraries)
        return tuple(libs)

    def tensor_specs(self):
        out = [TensorSpec(self.spec.table, (self.spec.vocab, self.spec.dim), "table")]
        for p in (self.project_in, self.position):
            if p is not None:
                out += p.tensor_specs()
        return out

    def load(self, tensors, device, act_dtype):
        self.table = weight_to_device(tensors[self.spec.table], device, act_dtype, self.spec.table)
        for p in (self.project_in, self.position):
            if p is not None:
                p.load(tensors, device, act_dtype)

    def parameter_bytes(self):
        n = self.table.numel() * self.table.element_size()
        for p in (self.project_in, self.position):
            if p is not None:
                n += p.parameter_bytes()
        return n

    def forward(self, ctx, x, x_act):
        """Fills x (32-bit) and, when given, x_act."""
        table_pos = self.position.table_for_embedding() if self.position is not None else None
        pos_table, offset = table_pos if table_pos is not None else (None, 0)
        if self.project_in is None:
            tok, pre = self.table, None
            if pos_table is not None and pos_table.dtype != tok.dtype:
                pos_table = pos_table.to(tok.dtype)
        else:
            e = ctx.empty(ctx.n_tokens, self.spec.dim)
            ops.gather_rows(self.table, ctx.token_ids, e)
            pre = ctx.empty(ctx.n_tokens, x.shape[1], torch.float32)
            self.project_in.forward(e, pre)
            tok = None
        freq = getattr(self.position, "frequencies_for_embedding", lambda: None)() if self.position is not None else None
        ops.embed(tok, pre, ctx.token_ids, pos_table, ctx.positions, offset, x, x_act, tok_scale=self.spec.scale,
                  sin_freq=freq)
        if self.position is not None and table_pos is None and freq is None:
            self.position.embed(ctx, x)
            if x_act is not None:
                ops.pick_rows(x, None, out_act=x_act)


class StreamJoin(Part):
    """x <- W [x; x0], x0 being the stream as the embedding left it, where the schedule asks for it.  W is kept as its two
    halves: x0's product does not change from one place to the next, so it is formed once a step (32-bit) and every join is
    one product of x with the other half, to which the epilogue adds it."""
    graph_safe = True

    def __init__(self, spec: StreamJoinSpec):
        s = self.spec = spec
        if s.weight.in_features != 2 * s.weight.out_features or s.weight.bias:
            raise ValueError("a join's matrix is [hidden, 2 hidden] and has no bias")
        self.stream = self.start = None

    @property
    def libraries(self):
        return ("gemm_simt", "gemm_tc", "gemv", "layernorm")        # the last: a copy of the stream in the activation type

    def tensor_specs(self):
        w = self.spec.weight
        return [TensorSpec(w.weight, (w.out_features, w.in_features), "matrix")]

    def load(self, tensors, device, act_dtype):
        name, H = self.spec.weight.weight, self.spec.weight.out_features
        w = weight_to_device(tensors[name], device, act_dtype, name)
        self.stream, self.start = w[:, :H].contiguous(), w[:, H:].contiguous()

    def parameter_bytes(self):
        return sum(w.numel() * w.element_size() for w in (self.stream, self.start))

    def begin(self, ctx, x0_act):
        """The part of every join that x0 alone decides."""
        out = ctx.carry(("join", self.spec), x0_act.shape[0], x0_act.shape[1], torch.float32)
        linear_forward(x0_act, self.start, None, out)
        return out

    def forward(self, ctx, x, x_act, from_start):
        """x <- W_x x_act + from_start (what begin() returned); x_act is x in the activation type, in memory of its own."""
        linear_forward(x_act, self.stream, None, x, residual=from_start)


class Head(Part):
    graph_safe = True
    def __init__(self, spec: HeadSpec):
        self.spec = spec
        self.weight = None
        self.final_norm = build_part("norm", spec.final_norm) if spec.final_norm else None
        self.project_out = Linear(spec.project_out) if spec.project_out else None
        if float(spec.logit_scale) != 1.0 and (self.final_norm is None or not getattr(self.final_norm, "takes_out_scale", False)):
            raise ValueError("a head that multiplies its logits by a constant needs a final norm whose kernel applies it")

    @property
    def libraries(self):
        libs = ["gemm_simt", "gemm_tc", "gemv"]
        # without a final norm the rows are picked by a kernel of the LayerNorm library
        libs += list(self.final_norm.libraries) if self.final_norm is not None else ["layernorm"]
        return tuple(dict.fromkeys(libs))

    def tensor_specs(self):
        s = self.spec
        out = [TensorSpec(s.weight, (s.vocab, s.dim), "matrix", tied_to=s.tied_to)]
        for p in (self.final_norm, self.project_out):
            if p is not None:
                out += p.tensor_specs()
        return out

    def load(self, tensors, device, act_dtype, shared=None):
        """`shared`: {tensor name: device tensor} of tensors another part already holds (the tied table)."""
        s = self.spec
        src = tensors[s.weight]
        if shared is not None and s.tied_to in shared and src is tensors.get(s.tied_to):
            self.weight = shared[s.tied_to]
        else:
            self.weight = weight_to_device(src, device, act_dtype, s.weight)
        for p in (self.final_norm, self.project_out):
            if p is not None:
                p.load(tensors, device, act_dtype)

    def parameter_bytes(self):
        n = self.weight.numel() * self.weight.element_size()
        for p in (self.final_norm, self.project_out):
            if p is not None:
                n += p.parameter_bytes()
        return n

    def forward(self, ctx, x, rows) -> torch.Tensor:
        """32-bit logits [len(rows), vocab] of the picked rows of the residual stream."""
        R = rows.shape[0]
        y = ctx.empty(R, x.shape[1])
        scale = float(self.spec.logit_scale)
        if self.final_norm is not None and scale != 1.0:
            # the constant rides on the norm's 32-bit output: the product that follows is linear
            self.final_norm.forward(ctx, x, out_act=y, rows=rows, out_scale=scale)
        elif self.final_norm is not None:
            self.final_norm.forward(ctx, x, out_act=y, rows=rows)
        else:
            ops.pick_rows(x, rows, out_act=y)
        if self.project_out is not None:
            z = ctx.empty(R, self.spec.dim)
            self.project_out.forward(y, z)
            y = z
        logits = torch.empty((R, self.spec.vocab), dtype=torch.float32, device=ctx.device)
        linear_forward(y, self.weight, None, logits)
        return logits
