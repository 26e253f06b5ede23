"""The Resatar architecture as data: its configuration -> a ModelSpec naming parts, sizes, constants and tensors.

A decoder whose layers are listed one by one in the configuration, with a norm before and behind every sublayer:
x <- x + n1b(mixer(n1(x))), x <- x + n2b(ff(n2(x))); every norm of the stream is an RMS norm with ONE learned number.
Three mixers:

  attention   softmax attention rotated by position with frequencies stretched by their wave length; a layer with v_mix
              mixes its values with those of the first such layer (the same tokens'); one output gate per head
  mamba1      a selective scan with a decay per channel and state, behind a short causal convolution
  parallel    two mixers on the same input, each with a factor: softmax attention without rotation (queries and keys
              normalised over the whole projection, a logarithmic distance bias taken off the scores, a sliding window
              that keeps the first tokens, a gate per element), and linear attention with a fixed decay per head
              behind silu projections, normalised over all heads together and gated

The feed-forward is down(gelu(up h)), or routed experts down(silu(gate h) * up h) whose weights are the softmax of the
chosen logits, plus a shared expert that every token runs.  The head is a matrix of its own behind a final norm.

Tensor names: 'embed', 'final.norm', 'head', and for layer i the prefix 'l<i>.': 'norm1', 'norm1b', 'norm2', 'norm2b',
'mlp.up|down' or 'mlp.router', 'mlp.router.b', 'mlp.e<j>.gate|up|down', 'mlp.shared.gate|up|down', and under 'mix.':
q, k, v, vmix, g, o | in, conv, conv.b, x, dt, dt.b, A_log, D, o | left.q, left.q.b, left.k, left.k.b, left.v, left.v.b,
left.q.norm, left.k.norm, left.r1, left.r2, left.g, left.o, left.o.b, right.q, right.k, right.v, right.g, right.norm,
right.o.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.resatar_config import ResatarConfig
from ..parts.spec import (DenseFeedForwardSpec, EmbeddingSpec, ExpertSpec, FrequencyBandsSpec, GatedFeedForwardSpec, HeadSpec,
                          LayerSpec, LinearSpec, ModelSpec, NormSpec, ParallelMixerSpec, RetentionSpec, RotaryAttentionSpec,
                          RotarySpec, RoutedFeedForwardSpec, ScheduleEntry, SelectiveScanSpec)


def _lin(name: str, n_in: int, n_out: int, bias: bool = False) -> LinearSpec:
    return LinearSpec(n_in, n_out, name, name + ".b" if bias else None)


def _attention(p: str, W: int, m: dict, eps: float, i: int, first) -> RotaryAttentionSpec:
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot")
    sc = rot.get("scaling") if rot else None
    mixes = bool(m["v_mix"])
    return RotaryAttentionSpec(
        kind="rotary_attention", hidden=W, n_heads=H, n_kv_heads=G, k_dim=d, v_dim=dv, scale=float(m["scale"]),
        q=_lin(p + ".q", W, H * d), k=_lin(p + ".k", W, G * d), v=_lin(p + ".v", W, G * dv), out=_lin(p + ".o", H * dv, W),
        rotary=RotarySpec(rot["dims"], float(rot["base"]), scaling=FrequencyBandsSpec(
            float(sc["factor"]), float(sc["low"]), float(sc["high"]), float(sc["original"])) if sc else None) if rot else None,
        gate=_lin(p + ".g", W, H), gate_per_head=True,
        value_mix=p + ".vmix" if mixes else None, value_source=first if mixes and i != first else None)


def _selective_scan(p: str, W: int, m: dict) -> SelectiveScanSpec:
    C, R, N = m["inner"], m["dt_rank"], m["state"]
    return SelectiveScanSpec(kind="selective_scan", hidden=W, inner=C, state=N, dt_rank=R, conv_taps=m["conv"],
                             in_proj=_lin(p + ".in", W, 2 * C), x_proj=_lin(p + ".x", C, R + 2 * N),
                             dt_proj=_lin(p + ".dt", R, C, True), out=_lin(p + ".o", C, W), conv=p + ".conv",
                             conv_bias=p + ".conv.b", a_log=p + ".A_log", skip=p + ".D",
                             activation="silu")


def _parallel(p: str, W: int, m: dict, eps: float) -> ParallelMixerSpec:
    l, r = m["left"], m["right"]
    H, G, d, dv = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
    mask, pl, pr = l.get("mask"), p + ".left", p + ".right"
    left = RotaryAttentionSpec(
        kind="rotary_attention", hidden=W, n_heads=H, n_kv_heads=G, k_dim=d, v_dim=dv, scale=float(l["scale"]),
        q=_lin(pl + ".q", W, H * d, True), k=_lin(pl + ".k", W, G * d, True), v=_lin(pl + ".v", W, G * dv, True),
        out=_lin(pl + ".o", H * dv, W, True), q_norm=pl + ".q.norm", k_norm=pl + ".k.norm", norm_eps=eps,
        distance_mul=pl + ".r1", distance_rate=pl + ".r2", gate=_lin(pl + ".g", W, H * dv),
        window=mask["size"] if mask else None, keep_first=mask["keep_first"] if mask else 0)
    H, d, dv = r["heads"], r["dim"], r["vdim"]
    right = RetentionSpec(
        kind="retention", hidden=W, n_heads=H, k_dim=d, v_dim=dv, decay=tuple(float(x) for x in r["decay"]),
        q=_lin(pr + ".q", W, H * d), k=_lin(pr + ".k", W, H * d), v=_lin(pr + ".v", W, H * dv),
        gate=_lin(pr + ".g", W, H * dv), out=_lin(pr + ".o", H * dv, W), norm_eps=eps, activation="silu",
        gate_activation="sigmoid", joint_norm=True, out_norm=pr + ".norm")
    return ParallelMixerSpec(kind="parallel", branches=(left, right), scales=(float(m["left_scale"]), float(m["right_scale"])))


def _gated(p: str, W: int, F: int) -> GatedFeedForwardSpec:
    return GatedFeedForwardSpec(kind="gated_dense", gate=_lin(p + ".gate", W, F), up=_lin(p + ".up", W, F),
                                down=_lin(p + ".down", F, W), activation="silu")


def _feed_forward(p: str, W: int, mlp: dict):
    if mlp["kind"] == "dense":
        F = mlp["ff"]
        return DenseFeedForwardSpec(kind="dense", fc1=_lin(p + ".up", W, F), fc2=_lin(p + ".down", F, W), activation="gelu_new")
    r, shared = mlp["router"], mlp.get("shared")
    return RoutedFeedForwardSpec(
        kind="routed_experts", hidden=W, ff=mlp["expert"]["ff"], n_experts=r["experts"], top=r["top"], router=p + ".router",
        router_bias=p + ".router.b",
        experts=tuple(ExpertSpec(f"{p}.e{j}.gate", f"{p}.e{j}.up", f"{p}.e{j}.down") for j in range(r["experts"])),
        # the softmax over all logits, renormalised over the chosen ones, is the softmax over the chosen logits
        scores="softmax", renormalize=True, weight_on_input=False, act_alpha=1.0, up_shift=0.0,
        shared=_gated(p + ".shared", W, shared["ff"]) if shared else None)


def build_spec(cfg: ResatarConfig) -> ModelSpec:
    W, eps, first = cfg.width, cfg.norm_eps, cfg.first_mixing_layer
    norm = lambda name: NormSpec("rms_norm", W, eps, weight=name, one_number=True)
    layers = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}", layer["mixer"]
        if layer["type"] == "attention":
            mixer = _attention(p + ".mix", W, m, eps, i, first)
        elif layer["type"] == "mamba1":
            mixer = _selective_scan(p + ".mix", W, m)
        else:
            mixer = _parallel(p + ".mix", W, m, eps)
        ff = n2 = n2b = None
        if layer.get("mlp") is not None:
            ff, n2, n2b = _feed_forward(p + ".mlp", W, layer["mlp"]), norm(p + ".norm2"), norm(p + ".norm2b")
        layers.append(LayerSpec(block="sandwich_norm", norm1=norm(p + ".norm1"), mixer=mixer, norm1_post=norm(p + ".norm1b"),
                                norm2=n2, feed_forward=ff, norm2_post=n2b))
    # a layer's cache number is its index: a layer that mixes in another's values names that layer
    return ModelSpec(hidden_size=W, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
                     embedding=EmbeddingSpec(table="embed", vocab=cfg.vocab, dim=W), layers=tuple(layers),
                     schedule=tuple(ScheduleEntry(i, i) for i in range(len(layers))),
                     head=HeadSpec(weight="head", vocab=cfg.vocab, dim=W, final_norm=norm("final.norm")))


register_architecture(Architecture(name="Resatar", model_type="resatar", config_class=ResatarConfig, build_spec=build_spec))
