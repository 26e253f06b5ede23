"""A decoder put together from parts according to a ModelSpec: embedding, the scheduled layers,
head.  It knows no architecture: models/opt.py (or a test) supplies the specification."""
from __future__ import annotations

import contextlib
from typing import Dict, List, Optional

import torch

from ..kernels import build as kbuild
from ..kernels import ops
from ..parts import Embedding, Head, StreamJoin, build_block, build_part
from ..parts.spec import ModelSpec
from ..weights.loader import TensorSpec


class DecoderModel:
    def __init__(self, spec: ModelSpec):
        self.spec = spec
        self.embedding = Embedding(spec.embedding)
        self.blocks = []
        for ls in spec.layers:
            self.blocks.append(build_block(ls.block, build_part("norm", ls.norm1), build_part("mixer", ls.mixer),
                                           build_part("norm", ls.norm2),
                                           build_part("feed_forward", ls.feed_forward), layer_spec=ls))
        self.joins = {j: StreamJoin(j) for j in dict.fromkeys(e.join for e in spec.schedule) if j is not None}
        self.head = Head(spec.head)
        for e in spec.schedule:
            if not (0 <= e.layer < len(self.blocks)):
                raise ValueError(f"schedule names layer {e.layer}, the model has {len(self.blocks)}")
        for j in self.joins:
            if j.weight.out_features != spec.hidden_size:
                raise ValueError(f"a join of width {j.weight.out_features} in a model of width {spec.hidden_size}")
        self.device = None
        self.act_dtype = None
        self._taps: Optional[Dict[str, torch.Tensor]] = None

    # ---- taps -----------------------------------------------------------------------------------
    @contextlib.contextmanager
    def tap_hidden_states(self):
        """Inside the block every step leaves copies of its intermediate results in the dictionary
        that is yielded: "embedding", "entry<i>" (the 32-bit residual stream [tokens, hidden] after
        the i-th schedule entry) and "logits"; a later step overwrites them.  Steps run eagerly
        meanwhile (a captured graph would write into buffers of its own).  The counterpart of the
        reference's named debug tensors (src/transformers_neuronx/global_debugger.py:27-91)."""
        taps: Dict[str, torch.Tensor] = {}
        prev, self._taps = self._taps, taps
        try:
            yield taps
        finally:
            self._taps = prev

    # ---- parts, tensors, kernels --------------------------------------------------------------
    def all_parts(self):
        out = [self.embedding]
        for b in self.blocks:
            out += b.parts()
        out += list(self.joins.values())
        out.append(self.head)
        return out

    def tensor_specs(self) -> List[TensorSpec]:
        seen, out = set(), []
        for p in self.all_parts():
            for s in p.tensor_specs():
                if s.name not in seen:
                    seen.add(s.name)
                    out.append(s)
        return out

    def libraries(self, act_dtype=None) -> List[str]:
        """Kernel libraries worth compiling before the first step (the rest are compiled when first used)."""
        libs = []
        for p in self.all_parts():
            libs += [l for l in p.libraries if l in kbuild.SOURCES]
        if act_dtype == torch.float32:
            libs = [l for l in libs if l not in ("gemm_tc", "gemv", "attention_prefill", "attention_prefill_tc", "attention_decode",
                                                 "moe_grouped")]
        return list(dict.fromkeys(libs))

    @property
    def graph_safe(self) -> bool:
        """Whether a step of this model can be captured in a CUDA graph now (every part says so,
        and nobody is tapping intermediate results)."""
        return self._taps is None and all(getattr(p, "graph_safe", False) for p in self.all_parts())

    def cache_needs(self) -> Dict[int, object]:
        """{cache id -> what the mixer(s) using it keep}; entries sharing a cache must agree."""
        needs: Dict[int, object] = {}
        for e in self.spec.schedule:
            need = self.blocks[e.layer].mixer.cache_need()
            # a mixer that keeps several things (say pages of keys and values and a recurrent state) returns a
            # tuple of needs: they become the caches (entry's cache, 0), (entry's cache, 1), ...
            several = isinstance(need, (tuple, list))
            for j, nd in enumerate(need if several else (need,)):
                cid = (e.cache, j) if several else e.cache
                if cid in needs and needs[cid] != nd:
                    raise ValueError(f"cache {cid} is shared by mixers with different needs: {needs[cid]} and {nd}")
                needs[cid] = nd
        return needs

    def load(self, tensors: Dict[str, torch.Tensor], device, act_dtype) -> None:
        self.device, self.act_dtype = device, act_dtype
        self.embedding.load(tensors, device, act_dtype)
        for b in self.blocks:
            for p in b.parts():
                p.load(tensors, device, act_dtype)
        for j in self.joins.values():
            j.load(tensors, device, act_dtype)
        self.head.load(tensors, device, act_dtype, shared={self.spec.embedding.table: self.embedding.table})

    def parameter_bytes(self) -> int:
        """Bytes of every weight one step reads once (a tied table counted once)."""
        n, seen = 0, set()
        for p in self.all_parts():
            n += p.parameter_bytes()
        if self.head.weight is self.embedding.table:
            n -= self.head.weight.numel() * self.head.weight.element_size()
        return n

    # ---- one step -------------------------------------------------------------------------------
    def forward(self, ctx) -> torch.Tensor:
        """Runs the tokens of ctx through the scheduled layers; returns 32-bit logits of ctx.logit_rows
        ([0, vocab] when none is wanted)."""
        N, H = ctx.n_tokens, self.spec.hidden_size
        x = ctx.empty(N, H, torch.float32)
        schedule, joins = self.spec.schedule, self.joins
        first = self.blocks[schedule[0].layer] if schedule else None
        want_act = any(self.blocks[e.layer].needs_act_input for e in schedule)
        x_act = ctx.empty(N, H) if (want_act or joins) else None
        act_current = first is not None and (first.needs_act_input or bool(joins))       # x_act holds x
        self.embedding.forward(ctx, x, x_act if act_current else None)
        from_start = {j: part.begin(ctx, x_act) for j, part in joins.items()}
        taps = self._taps
        ctx.handed_on = None
        if taps is not None:
            taps.clear()
            taps["embedding"] = x.clone()
        for i, e in enumerate(schedule):
            block = self.blocks[e.layer]
            if e.join is not None:
                if not act_current:
                    ops.pick_rows(x, None, out_act=x_act)
                joins[e.join].forward(ctx, x, x_act, from_start[e.join])
                act_current = False
            if block.needs_act_input and not act_current:
                ops.pick_rows(x, None, out_act=x_act)
            ctx.cache_id = e.cache
            ctx.entry_index = i
            after = schedule[i + 1] if i + 1 < len(schedule) else None
            # nothing can be prepared for a block whose input a join still changes; the join wants the stream's copy
            ctx.next_block = self.blocks[after.layer] if after is not None and after.join is None else None
            ctx.stream_copy = x_act if after is not None and after.join is not None and not block.needs_act_input else None
            wanted = ctx.stream_copy is not None
            ctx.begin_entry()
            block.forward(ctx, x, x_act)
            act_current = block.keeps_act_current or (wanted and ctx.stream_copy is None)
            if taps is not None:
                taps[f"entry{i}"] = x.clone()
        if ctx.logit_rows is None or ctx.logit_rows.shape[0] == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32, device=ctx.device)
        logits = self.head.forward(ctx, x, ctx.logit_rows)
        if taps is not None:
            taps["logits"] = logits.clone()
        return logits
