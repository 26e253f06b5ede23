"""The Taborax architecture as data: its configuration -> a ModelSpec naming parts, sizes, constants and tensors.

A decoder whose layers are listed one by one in the configuration.  Every sublayer has a norm before it and one behind it:
x <- x + norm1b(mixer(norm1(x))), then x <- x + norm2b(ff(norm2(x))), RMS norms with plain weights.  A run of layers may be
looped: it is walked several times with the same weights, every pass with a cache of its own, and ahead of each pass the
stream is joined with the embedding output, x <- W_in [x; x0].  Here that is a schedule which names those layers several
times with different cache numbers, the first of each pass with a join.

  latent_attention  queries through a normalised latent; keys and values expanded per head from one normalised latent, which
                    is all the pages hold; no positions
  attention         grouped key/value heads, q and k rotated in halves over the first rot.dims dims; the values are the keys
                    as projected; every softmax shares its weight with an empty key of score 0 (a sink)

The feed-forward is down(relu(up h)^2), or routed experts: softmax scores over experts and identity experts together, a
correction of the choice, groups scored by their best expert, weights that are the scores as they are, and a shared expert
behind a gate.  The head is a matrix of its own behind a final norm.

Tensor names: 'embed', 'loop.in', 'final.norm', 'head', and for layer i the prefix 'l<i>.': 'norm1', 'norm1b', 'norm2',
'norm2b', under 'mix.': dq, dq.norm, uq, dkv, dkv.norm, uk, uv, o | q, k, o, and under 'mlp.': up, down | router, correction,
e<j>.gate|up|down, shared.gate|up|down|sg.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.taborax_config import TaboraxConfig
from ..parts.spec import (DenseFeedForwardSpec, EmbeddingSpec, ExpertSpec, GatedFeedForwardSpec, HeadSpec,
                          LatentAttentionSpec, LayerSpec, LinearSpec, ModelSpec, NormSpec, RotaryAttentionSpec, RotarySpec,
                          RoutedFeedForwardSpec, ScheduleEntry, StreamJoinSpec)

SINK_SCORE = 0.0               # exp(0): the one in the softmax's denominator


def _lin(name: str, n_in: int, n_out: int) -> LinearSpec:
    return LinearSpec(n_in, n_out, name)


def _attention(p: str, W: int, m: dict, eps: float) -> RotaryAttentionSpec:
    H, G, d, rot = m["heads"], m["kv_heads"], m["dim"], m.get("rot")
    rotary = RotarySpec(rot["dims"], float(rot["base"])) if rot and rot.get("dims") else None
    return RotaryAttentionSpec(kind="rotary_attention", hidden=W, n_heads=H, n_kv_heads=G, k_dim=d, v_dim=d,
                               scale=float(m["scale"]), q=_lin(p + ".q", W, H * d), k=_lin(p + ".k", W, G * d), v=None,
                               out=_lin(p + ".o", H * d, W), rotary=rotary, sink=SINK_SCORE)


def _latent(p: str, W: int, m: dict, eps: float) -> LatentAttentionSpec:
    H, d, dv, rq, rkv = m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"]
    return LatentAttentionSpec(kind="latent_attention", hidden=W, n_heads=H, k_dim=d, rot_dim=0, v_dim=dv, q_rank=rq,
                               kv_rank=rkv, scale=float(m["scale"]), dq=_lin(p + ".dq", W, rq), uq=_lin(p + ".uq", rq, H * d),
                               dkv=_lin(p + ".dkv", W, rkv), uk=p + ".uk", uv=p + ".uv", out=_lin(p + ".o", H * dv, W),
                               q_norm=p + ".dq.norm", kv_norm=p + ".dkv.norm", norm_eps=eps)


_MIXERS = {"attention": _attention, "latent_attention": _latent}


def _feed_forward(p: str, W: int, mlp: dict):
    if mlp["kind"] == "dense":
        F = mlp["ff"]
        return DenseFeedForwardSpec(kind="dense", fc1=_lin(p + ".up", W, F), fc2=_lin(p + ".down", F, W), activation="relu2")
    r, groups, shared = mlp["router"], mlp["router"].get("groups"), mlp.get("shared")
    E, S = r["experts"], shared["ff"] if shared else 0
    return RoutedFeedForwardSpec(
        kind="routed_experts", hidden=W, ff=mlp["expert"]["ff"], n_experts=E, n_identity=r.get("identity") or 0, top=r["top"],
        router=p + ".router", correction=p + ".correction",
        experts=tuple(ExpertSpec(f"{p}.e{j}.gate", f"{p}.e{j}.up", f"{p}.e{j}.down") for j in range(E)),
        scores="softmax", renormalize=False, weight_on_input=False, act_alpha=1.0, up_shift=0.0,
        n_groups=groups["count"] if groups else 1, keep_groups=groups["keep"] if groups else 1, group_top=1,
        shared=GatedFeedForwardSpec(kind="gated_dense", gate=_lin(p + ".shared.gate", W, S), up=_lin(p + ".shared.up", W, S),
                                    down=_lin(p + ".shared.down", S, W), activation="silu") if shared else None,
        shared_gate=p + ".shared.sg" if shared else None)


def build_spec(cfg: TaboraxConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    norm = lambda name: NormSpec("rms_norm", W, eps, weight=name)
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}"
        ff = n2 = n2b = None
        if layer.get("mlp") is not None:
            ff, n2, n2b = _feed_forward(p + ".mlp", W, layer["mlp"]), norm(p + ".norm2"), norm(p + ".norm2b")
        layers.append(LayerSpec(block="sandwich_norm", norm1=norm(p + ".norm1"),
                                mixer=_MIXERS[layer["type"]](p + ".mix", W, layer["mixer"], eps), norm2=n2,
                                feed_forward=ff, norm1_post=norm(p + ".norm1b"), norm2_post=n2b))
    # every run of a layer is a schedule entry with a cache of its own: a looped layer keeps one past per pass
    join = StreamJoinSpec(_lin("loop.in", 2 * W, W))
    schedule = tuple(ScheduleEntry(layer, run, join if begins else None) for run, (layer, begins) in enumerate(cfg.layer_runs()))
    return ModelSpec(hidden_size=W, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
                     embedding=EmbeddingSpec(table="embed", vocab=cfg.vocab, dim=W), layers=tuple(layers), schedule=schedule,
                     head=HeadSpec(weight="head", vocab=cfg.vocab, dim=W, final_norm=norm("final.norm")))


register_architecture(Architecture(name="Taborax", model_type="taborax", config_class=TaboraxConfig, build_spec=build_spec))
