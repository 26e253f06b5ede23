"""Shared by the Resatar tests: small configurations that differ from one another in every size and constant (head counts
and shared key/value heads, key and value sizes that are and are not padded, partly rotated heads with and without
stretched frequencies, with and without mixed values, windows with and without kept first tokens, recurrences of many
shapes, one to eight taps, dense and routed feed-forwards with and without a shared expert, layers without a
feed-forward), and a model folder with seeded random weights beside the plain implementation's answers
(tests/plain/resatar_plain.py)."""
from __future__ import annotations

import torch

from plain import resatar_plain as RP
from vononex_helpers import TOLERANCE, VononexModel, cut_steps, mixed_steps, whole_steps  # noqa: F401
from vozirax_helpers import compare, layer  # noqa: F401


def rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def attn(heads, kv, dim, vdim, scale, rotary=None, v_mix=False):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if rotary is not None:
        m["rot"] = rotary
    return m


def mamba(inner, dt_rank, state, conv):
    return {"inner": inner, "dt_rank": dt_rank, "state": state, "conv": conv}


def left(heads, kv, dim, vdim, scale, mask=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if mask is not None:
        m["mask"] = {"size": mask[0], "keep_first": mask[1]}
    return m


def right(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def side(l, r, ls, rs):
    return {"left": l, "right": r, "left_scale": ls, "right_scale": rs}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


# Odd sizes everywhere: heads of 20 dims of which 12 turn, values of 28 (padded to 32), stretched and plain frequencies, values
# mixed from two layers on (a layer between them that neither mixes nor turns), a window of 23 that keeps 5, no window,
# a state of 18 behind five taps, recurrent heads of 18 x 10, a shared expert as wide as no expert and none, two
# layers without a feed-forward, widths the tensor-core product refuses.
CONFIG_A = {"architecture": "Resatar", "vocab": 211, "width": 72, "norm": {"eps": 1e-4}, "init_std": 0.2,
            "layers": [
                layer("attention", attn(6, 2, 20, 28, 0.3, rot(12, 1e4, (8.0, 1.5, 6.0, 64)), True), moe(6, 3, 20, 28)),
                layer("mamba1", mamba(60, 5, 18, 5), None),
                layer("parallel", side(left(6, 3, 12, 20, 0.35, (23, 5)), right(5, 18, 10, (0.5, 0.9, 0.99, 0.999, 0.7)), 0.7, -1.3),
                      dense(88)),
                layer("attention", attn(3, 3, 8, 24, 0.4), dense(50)),
                layer("attention", attn(4, 2, 16, 28, 0.25, rot(16, 500.0), True), moe(5, 1, 36)),
                layer("parallel", side(left(2, 2, 24, 12, 0.2), right(1, 4, 30, (0.97,)), 1.4, 0.9), None),
                layer("attention", attn(2, 2, 24, 28, 0.2, rot(20, 2e3, (3.0, 1.0, 2.0, 40)), True), dense(40))]}
# Sizes the tensor-core kernels take: heads of 64, 96 and 128, a window of 72 that keeps 20 (so that whole tiles and pages lie
# between them), recurrent heads of 128 x 64, a state of 16 behind four taps, a shared expert as wide as the experts and one that
# is not.
CONFIG_B = {"architecture": "Resatar", "vocab": 1003, "width": 256, "norm": {"eps": 1e-6}, "init_std": 0.1,
            "layers": [
                layer("mamba1", mamba(384, 16, 16, 4), dense(512)),
                layer("attention", attn(8, 2, 64, 64, 0.12, rot(32, 1e5, (4.0, 1.0, 4.0, 128)), True), moe(8, 2, 128, 128)),
                layer("parallel", side(left(8, 2, 128, 128, 0.3, (72, 20)), right(4, 128, 64, (0.6, 0.9, 0.99, 0.9995)), 1.1, 0.6),
                      moe(4, 2, 96, 160)),
                layer("attention", attn(4, 2, 96, 64, 0.1, rot(96, 1e4, (2.0, 1.0, 8.0, 96)), True), None)]}
# A width and a vocabulary that are no multiples of 8 (the 16-bit engine falls back to the CUDA-core product and to scalar
# loads), one head, windows of 1 and of 16 that keeps 17, states of 70 and 3, one and eight taps, a step rank of 1, an expert alone.
CONFIG_C = {"architecture": "Resatar", "vocab": 333, "width": 100, "norm": {"eps": 1e-5}, "init_std": 0.2,
            "layers": [
                layer("parallel", side(left(1, 1, 50, 30, 0.14, (16, 17)), right(3, 7, 9, (0.9, 0.2, 0.999)), 1.0, 1.0),
                      moe(1, 1, 24, 24)),
                layer("mamba1", mamba(50, 1, 70, 1), dense(36)),
                layer("attention", attn(5, 5, 8, 20, 0.3, rot(4, 1e4), True), moe(4, 4, 28)),
                layer("mamba1", mamba(30, 7, 3, 8), None),
                layer("parallel", side(left(4, 2, 16, 16, 0.5, (1, 0)), right(2, 30, 20, (0.95, 0.8)), 0.5, 2.0), dense(44))]}
CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C}


class ResatarModel(VononexModel):
    def plain_logits(self, ids):
        key = tuple(int(i) for i in ids)
        if key not in self._cache:
            self._cache[key] = RP.forward(self.cfg_dict, self.plain_tensors, list(key)).float()
        return self._cache[key]

    def plain_hidden(self, ids):
        return torch.stack(RP.forward(self.cfg_dict, self.plain_tensors, [int(i) for i in ids], keep_layers=True)[1]).float()
