"""Shared by the Taborax tests: small configurations that differ from one another in every size and constant (head counts
and shared key heads, latents narrower and wider than the heads, partly, wholly and un-rotated heads, routers with one
group and several, with and without identity experts, shared experts of the experts' width, of a multiple and of neither,
loops over one layer, over several and none, layers without a feed-forward), and a model folder with seeded random weights
beside the plain implementation's answers (tests/plain/taborax_plain.py)."""
from __future__ import annotations

import torch

from plain import taborax_plain as BP
from vononex_helpers import TOLERANCE, VononexModel, cut_steps, mixed_steps, whole_steps  # noqa: F401
from vozirax_helpers import compare  # noqa: F401  (rows whose expert rounding decides are few and counted)


def latent(heads, dim, vdim, q_rank, kv_rank, scale):
    return {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}


def attn(heads, kv, dim, scale, rot_dims=0, base=1e4):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale}
    if rot_dims:
        m["rot"] = {"dims": rot_dims, "base": base}
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=0, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp):
    return {"type": "latent_attention" if "kv_rank" in mixer else "attention", "mixer": mixer, "mlp": mlp}


# Odd sizes everywhere: 5 heads of 12 over a latent of 40, values of 20; 6 heads on 2 key heads of 20 with 12 dims turned;
# 7 experts and 2 identity experts in three groups of which two are kept, a shared expert twice as wide as the others; a loop
# of three passes over two layers that begins behind the first layer; a layer without a feed-forward; no shared expert.
CONFIG_A = {"architecture": "Taborax", "vocab": 211, "width": 72, "norm": {"eps": 1e-4}, "init_std": 0.2,
            "loop": {"start": 1, "stop": 3, "times": 3}, "layers": [
                layer(latent(5, 12, 20, 28, 40, 0.3), moe(7, 3, 24, 2, (3, 2), 48)),
                layer(attn(6, 2, 20, 0.3, 12, 500.0), dense(88)),
                layer(latent(3, 30, 10, 9, 22, 0.2), None),
                layer(attn(2, 1, 64, 0.125, 64, 1e4), moe(4, 2, 36, 4, None, 30)),
                layer(attn(4, 4, 8, 0.5), moe(5, 2, 40, 1))]}
# Sizes the tensor-core kernels take: latents of 128 and 96, heads of 64, 128 and 80, 12 experts and 4 identity experts in
# four groups, a shared expert of the experts' width, of four times it and of neither; a loop over the whole model.
CONFIG_B = {"architecture": "Taborax", "vocab": 1003, "width": 256, "norm": {"eps": 1e-6}, "init_std": 0.1,
            "loop": {"start": 0, "stop": 4, "times": 2}, "layers": [
                layer(attn(8, 2, 128, 0.09, 64, 2e4), moe(12, 4, 64, 4, (4, 2), 64)),
                layer(latent(4, 64, 96, 72, 128, 0.12), moe(8, 1, 96, 0, (2, 1), 160)),
                layer(latent(6, 32, 64, 128, 96, 0.15), dense(384)),
                layer(attn(4, 4, 80, 0.11, 16, 1e5), moe(6, 2, 32, 2, None, 128))]}
# A width and a vocabulary that are no multiples of 8 (the 16-bit engine falls back to the CUDA-core product and to scalar
# loads), one head, one expert beside one identity expert, a group an expert, one pass of a loop, latents of 5 and 17.
CONFIG_C = {"architecture": "Taborax", "vocab": 333, "width": 100, "norm": {"eps": 1e-5}, "init_std": 0.2,
            "loop": {"start": 1, "stop": 2, "times": 1}, "layers": [
                layer(attn(1, 1, 50, 0.14, 10, 77.0), moe(1, 1, 20, 1, None, 20)),
                layer(latent(1, 7, 9, 3, 5, 0.4), moe(3, 2, 12, 3, (6, 4), 36)),
                layer(latent(5, 16, 16, 33, 17, 0.25), dense(36)),
                layer(attn(5, 5, 20, 0.22, 20, 2000.0), None)]}
# Rows wider than the 16-bit attention kernels take (256 dims a position), no loop.
CONFIG_D = {"architecture": "Taborax", "vocab": 120, "width": 96, "norm": {"eps": 1e-5}, "init_std": 0.1, "layers": [
                layer(latent(3, 24, 40, 20, 288, 0.2), moe(3, 3, 16, 2, None, 16)),
                layer(attn(2, 1, 272, 0.06, 32, 1e4), dense(64))]}
CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C, "D": CONFIG_D}


class TaboraxModel(VononexModel):
    def plain_logits(self, ids):
        key = tuple(int(i) for i in ids)
        if key not in self._cache:
            self._cache[key] = BP.forward_logits(key, self.plain_tensors, self.cfg_dict).float()
        return self._cache[key]

    def plain_hidden(self, ids):
        return BP.forward_hidden(tuple(int(i) for i in ids), self.plain_tensors, self.cfg_dict)[0].float()
