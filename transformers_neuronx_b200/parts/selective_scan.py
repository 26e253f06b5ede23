"""A selective state-space mixer with a decay per channel and state ("selective scan").

  W_in h = [x: inner | z: inner]
  x: one short causal convolution per channel over time (with bias), then an activation (silu)
  W_x x = [low: dt_rank | B: state | C: state];  dt = softplus(W_dt low + dt_bias), one per channel
  per channel c and state n:  S[c, n] <- exp(-exp(A_log[c, n]) dt_c) S[c, n] + dt_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c
  y * act(z); output projection

What the mixer keeps per request, both state of fixed size in the request's slot (zeroed when a request takes it): S
(inner x state) in 32-bit, and the last taps - 1 projected values of every convolved channel in the activation type, exactly
what a longer step would have read from its own rows.  Products and the convolution with its activation are in the
activation type, except that W_dt's product (with its bias) stays 32-bit; softplus, decays, state and y are 32-bit.  A step's tokens of
one request are walked in order by one kernel, portions of prompts and single tokens alike, so the state after a token does
not depend on how the prompt was cut.
"""
from __future__ import annotations

import math

import torch

from ..cache.manager import FixedStateNeed
from ..kernels import ops
from ..kernels.ops import activation_code
from ..weights.loader import TensorSpec
from .base import Mixer, to_device
from .fusable import pitched
from .linear import Linear
from .registry import register_mixer
from .spec import SelectiveScanSpec

MAX_TAPS = 8           # csrc/selective_scan.cu
MAX_STATE = 256


class SelectiveScan(Mixer):
    graph_safe = True
    can_overwrite = True
    libraries = ("gemm_simt", "gemm_tc", "gemv", "selective_scan", "conv_qkv")

    def __init__(self, spec: SelectiveScanSpec):
        s = self.spec = spec
        if not (1 <= s.conv_taps <= MAX_TAPS):
            raise ValueError(f"a convolution of {s.conv_taps} taps is not supported (1 to {MAX_TAPS})")
        if s.state > MAX_STATE:
            raise ValueError(f"state size {s.state} is not supported: the scan takes up to {MAX_STATE} numbers a channel")
        activation_code(s.activation)
        self.keep = s.conv_taps - 1
        self.in_proj, self.x_proj, self.dt_proj, self.out = (Linear(p) for p in (s.in_proj, s.x_proj, s.dt_proj, s.out))
        self.conv_w = self.conv_b = self.decay_log2 = self.skip = None

    def tensor_specs(self):
        s = self.spec
        out = []
        for p in (self.in_proj, self.x_proj, self.dt_proj, self.out):
            out += p.tensor_specs()
        out.append(TensorSpec(s.conv, (s.inner, s.conv_taps), "matrix"))
        if s.conv_bias:
            out.append(TensorSpec(s.conv_bias, (s.inner,), "bias"))
        out += [TensorSpec(s.a_log, (s.inner, s.state), "matrix")]
        if s.skip:
            out.append(TensorSpec(s.skip, (s.inner,), "bias"))
        return out

    def load(self, tensors, device, act_dtype):
        s = self.spec
        for p in (self.in_proj, self.x_proj, self.dt_proj, self.out):
            p.load(tensors, device, act_dtype)
        f32 = lambda name: to_device(tensors[name], device, torch.float32) if name else None
        self.conv_w = f32(s.conv).t().contiguous()            # [taps, channels]: a tap's weights of consecutive channels together
        self.conv_b, self.skip = f32(s.conv_bias), f32(s.skip)
        # the kernel's decay is 2^(decay_log2 * dt)
        self.decay_log2 = (-torch.exp(tensors[s.a_log].to(torch.float64)) / math.log(2.0)).to(torch.float32).to(device)

    def parameter_bytes(self):
        n = sum(p.parameter_bytes() for p in (self.in_proj, self.x_proj, self.dt_proj, self.out))
        return n + sum(t.numel() * 4 for t in (self.conv_w, self.conv_b, self.decay_log2, self.skip) if t is not None)

    def cache_need(self):
        s = self.spec
        state = FixedStateNeed((s.inner, s.state), "float32")
        if not self.keep:
            return (state,)
        return (state, FixedStateNeed((self.keep, s.inner), "activation"))

    def forward(self, ctx, h, out, accumulate=True):
        s, N = self.spec, h.shape[0]
        C, R, Ns = s.inner, s.dt_rank, s.state
        proj = pitched(ctx, N, 2 * C)
        self.in_proj.forward(h, proj)
        x = ctx.scratch(N, C)
        ops.causal_conv(proj, 0, self.conv_w, self.conv_b, s.conv_taps, ctx.cache(1) if self.keep else None, ctx, s.activation, x)
        low = pitched(ctx, N, R + 2 * Ns)
        self.x_proj.forward(x, low)
        dt = ctx.scratch(N, C, torch.float32)
        self.dt_proj.forward(low[:, :R], dt)
        y = ctx.scratch(N, C)
        ops.selective_scan(x, dt, low, R, R + Ns, self.decay_log2, self.skip, proj[:, C:2 * C], ctx.cache(0), ctx,
                           s.activation, y)
        self.out.forward(y, out, residual=out if accumulate else None)


register_mixer("selective_scan", SelectiveScan)
