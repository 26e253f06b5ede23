"""Softmax attention over the paged cache with rotated queries, keys and (optionally) values.

  q = W_q h + b, k = W_k h + b, v = W_v h + b
  q, k: RMS norm over the WHOLE projection (all heads at once) where the spec names a weight, before rotation
  q, k: rotated by position on the first rotary.dims dims of each head (dim i with dim i + dims/2)
  score(i, j) = scale * head_scale[h] * <q_i, k_j> - r1[h] ln(1 + r2[h] (i - j)) (the distance bias where the spec names
      its two tensors), causal; with a window, the last `window` positions and the first `keep_first` ones; softmax in 32-bit
  sink: one more key of a fixed score and without a value, exp(sink) more in the softmax's denominator
  rotate_values: v_j is turned by its position j over all v_dim dims before it is cached, and each head's
      output at position i is turned back by i: the sum then holds the values turned by j - i
  value mixing: the cached values are (1 - lambda) v + lambda v', v' the same tokens' values as an earlier entry of the
      schedule projected them (that entry leaves its projections in a buffer that outlives it)
  gate: the heads' outputs times sigmoid(W_g h), one number per head or per element, before the output projection
  output projection with bias
  a spec without a value projection: the values are the keys as projected (bias included), before their norm and
      rotation; nothing more is computed for them, the same columns of the product are read twice

Queries/keys (k_dim) and values (v_dim) may differ in size.  The cache's pages and the attention kernels take
one head size, so q, k and v are written with D = max(k_dim, v_dim) rounded up to 16 dims a head, the rest zero:
zeros in q and k add nothing to a score, zeros in v give output columns that are dropped.  With k_dim = v_dim a
multiple of 16 (the usual case) nothing is padded, and the kernels are those of every other attention part:
tcgen05 prefill, split-KV decode with its own cache append, the 32-bit kernel in a 32-bit engine.  head_scale
is folded into q in 32-bit before q is rounded.
"""
from __future__ import annotations

import math

import torch

from ..cache.manager import PagedKVNeed
from ..kernels import ops
from ..weights.loader import TensorSpec
from .base import to_device
from .fusable import FusableMixer
from .linear import Linear
from .registry import register_mixer
from .rotary import inverse_frequencies
from .spec import RotaryAttentionSpec


class RotaryAttention(FusableMixer):
    @property
    def extra_libraries(self):
        # the prefill kernel of this head size only: tcgen05 for 64 .. 128, mma.sync for the others
        prefill = "attention_prefill_tc" if self.pad_dim in (64, 80, 96, 112, 128) else "attention_prefill"
        return ("rotary_qkv", "kv_cache", "attention_simt", prefill, "attention_decode")

    def __init__(self, spec: RotaryAttentionSpec):
        s = self.spec = spec
        if s.n_heads % s.n_kv_heads:
            raise ValueError(f"{s.n_heads} heads cannot share {s.n_kv_heads} key/value heads")
        self.pad_dim = -(-max(s.k_dim, s.v_dim) // 16) * 16
        if self.pad_dim > 768:                       # up to 256 on the 16-bit kernels, beyond that on the CUDA cores
            raise ValueError(f"head sizes {s.k_dim}/{s.v_dim} are not supported: the attention kernels take up to 768")
        if s.rotary is not None and (s.rotary.dims > s.k_dim or s.rotary.dims % 2):
            raise ValueError(f"{s.rotary.dims} rotated dims do not fit heads of {s.k_dim}")
        if s.rotate_values and (s.rotary is None or s.v_dim % 2):
            raise ValueError("rotated values need a rotation and an even value size")
        self.values_are_keys = s.v is None
        if self.values_are_keys and (s.v_dim != s.k_dim or s.rotate_values):
            raise ValueError("values that are the keys have the keys' size and are not rotated")
        self.inputs = [Linear(s.q), Linear(s.k)] + ([] if self.values_are_keys else [Linear(s.v)])
        if (s.distance_mul is None) != (s.distance_rate is None):
            raise ValueError("a distance bias needs both of its tensors")
        if s.keep_first and not s.window:
            raise ValueError("first tokens are kept beside a window; without one every position is visible")
        if s.sink is not None and not math.isfinite(s.sink):
            raise ValueError(f"the sink's score must be a finite number, got {s.sink}")
        if s.gate is not None:
            want = s.n_heads * (1 if s.gate_per_head else s.v_dim)
            if s.gate.out_features != want:
                raise ValueError(f"the gate has {s.gate.out_features} outputs, needs {want}")
            self.inputs.append(Linear(s.gate))
        if s.value_source is not None and s.value_mix is None:
            raise ValueError("values of another entry are mixed in by a weight (value_mix)")
        if s.value_mix is not None and (self.values_are_keys or s.rotate_values):
            raise ValueError("mixed values are projected ones and are not rotated")
        self.output = Linear(s.out)
        self.q_weight = self.k_weight = self.head_scale = self.inv_freq_qk = self.inv_freq_v = None
        self.bias = self.mix_weight = None

    @property
    def inner_width(self):
        return self.spec.n_heads * self.spec.v_dim

    def extra_tensor_specs(self):
        s, out = self.spec, []
        if s.q_norm:
            out.append(TensorSpec(s.q_norm, (s.n_heads * s.k_dim,), "norm_weight"))
        if s.k_norm:
            out.append(TensorSpec(s.k_norm, (s.n_kv_heads * s.k_dim,), "norm_weight"))
        if s.head_scale:
            out.append(TensorSpec(s.head_scale, (s.n_heads,), "norm_weight"))
        if s.distance_mul:
            out += [TensorSpec(n, (s.n_heads,), "positive") for n in (s.distance_mul, s.distance_rate)]
        if s.value_mix:
            out.append(TensorSpec(s.value_mix, (), "bias"))
        return out

    def load_extras(self, tensors, device, act_dtype):
        s = self.spec
        f32 = lambda name: to_device(tensors[name], device, torch.float32) if name else None
        self.q_weight, self.k_weight, self.head_scale = f32(s.q_norm), f32(s.k_norm), f32(s.head_scale)
        if s.rotary is not None and s.rotary.dims:
            self.inv_freq_qk = inverse_frequencies(s.rotary.dims, s.rotary.base, device, s.rotary.scaling)
        if s.rotate_values:
            self.inv_freq_v = inverse_frequencies(s.v_dim, s.rotary.base, device)
        if s.distance_mul:
            self.bias = (f32(s.distance_mul), f32(s.distance_rate))
        if s.value_source is not None:
            self.mix_weight = f32(s.value_mix).reshape(1)

    def extra_parameter_bytes(self):
        return sum(t.numel() * 4 for t in (self.q_weight, self.k_weight, self.head_scale) + (self.bias or ())
                   if t is not None)

    def cache_need(self):
        s = self.spec
        return PagedKVNeed(s.n_kv_heads, self.pad_dim, s.window, keep_first=s.keep_first)

    def _value_columns(self, col0):
        s = self.spec
        k_off = col0 + s.n_heads * s.k_dim
        return k_off if self.values_are_keys else k_off + s.n_kv_heads * s.k_dim

    def projection_buffer(self, ctx, rows):
        s = self.spec
        if s.value_mix is None or s.value_source is not None:
            return super().projection_buffer(ctx, rows)
        # later entries read this one's values from its projections, so these outlive the entry
        width = self.projection_width
        proj = ctx.carry(("projections", ctx.cache_id), rows, -(-width // 8) * 8)[:, :width]
        v0 = self._value_columns(0)
        ctx.values_of[ctx.cache_id] = proj[:, v0:v0 + s.n_kv_heads * s.v_dim]
        return proj

    def mix(self, ctx, proj, col0, inner_out, out_scale, sub=None):
        s, D, N = self.spec, self.pad_dim, proj.shape[0]
        H, G = s.n_heads, s.n_kv_heads
        if sub is not None and s.value_mix is not None:
            raise NotImplementedError("a branch of another mixer does not share its values")
        q, k, v = ctx.scratch(N, H * D), ctx.scratch(N, G * D), ctx.scratch(N, G * D)
        k_off, v_off = col0 + H * s.k_dim, self._value_columns(col0)
        other = None
        if s.value_source is not None:
            other = ctx.values_of.get(s.value_source)
            if other is None or tuple(other.shape) != (N, G * s.v_dim):
                raise ValueError(f"entry {s.value_source} left no values of {G} heads of {s.v_dim} dims in this step")
        ops.rotary_qkv_prep(proj, col0, k_off, v_off, ctx.token_request, ctx.positions, self.q_weight,
                            self.k_weight, s.norm_eps, self.head_scale, self.inv_freq_qk,
                            s.rotary.dims if s.rotary is not None else 0, self.inv_freq_v, q, k, v, H, G, s.k_dim,
                            s.v_dim, D, other_values=other, mix_weight=self.mix_weight)
        cache, g = ctx.cache(sub), ctx.cache_group(sub)
        gate = None
        if s.gate is not None:
            g0 = v_off + G * (s.k_dim if self.values_are_keys else s.v_dim)
            gate = proj[:, g0:g0 + s.gate.out_features]
        # heads that are neither padded, turned back, gated nor scaled go from the attention kernel straight to their place
        direct = (D == s.v_dim and self.inv_freq_v is None and gate is None and out_scale == 1.0
                  and inner_out.dtype == q.dtype and inner_out.stride(0) % 8 == 0 and inner_out.data_ptr() % 16 == 0)
        att = inner_out if direct else ctx.scratch(N, H * D)
        ops.attention(ctx, g, q, cache, att, H, s.scale, s.window or 0, new_kv=(k, v, ctx.slot_mapping[g]),
                      keep_first=s.keep_first, bias=self.bias, sink=s.sink)
        if not direct:
            ops.rotary_unrotate(att, ctx.token_request, ctx.positions, self.inv_freq_v, out_scale, inner_out, H, s.v_dim, D,
                                gate=gate)


register_mixer("rotary_attention", RotaryAttention)
