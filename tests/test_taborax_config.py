"""The Taborax configuration, its tensors, its caches and its schedule, and the plain implementation's own mechanisms,
without a GPU."""
import copy
import math

import pytest
import torch

from plain import taborax_plain as BP
from taborax_helpers import CONFIG_A, CONFIG_B, CONFIG_C, CONFIG_D, CONFIGS, TaboraxModel, moe


def _spec(d):
    from transformers_neuronx_b200.config import config_from_dict
    arch, cfg = config_from_dict(copy.deepcopy(d))
    return arch, cfg, arch.build_spec(cfg)


def test_the_architecture_is_found_by_its_single_name_and_round_trips():
    from transformers_neuronx_b200.config import TaboraxConfig, config_from_dict
    for d in CONFIGS.values():
        arch, cfg, spec = _spec(d)
        assert arch.name == "Taborax" and isinstance(cfg, TaboraxConfig)
        again = config_from_dict(cfg.to_dict())[1]
        assert again == cfg and again.to_dict()["layers"] == cfg.to_dict()["layers"] and again.loop == d.get("loop")
        assert spec.vocab_size == d["vocab"] and spec.hidden_size == d["width"] and len(spec.layers) == len(d["layers"])
        for l in spec.layers:
            assert l.block == "sandwich_norm" and l.norm1.eps == d["norm"]["eps"] and l.norm1.weight_offset == 0.0


def test_tensor_names_and_shapes_follow_the_layers():
    from transformers_neuronx_b200.models.decoder import DecoderModel
    t = {s.name: tuple(s.shape) for s in DecoderModel(_spec(CONFIG_A)[2]).tensor_specs()}
    assert t["embed"] == (211, 72) == t["head"] and t["final.norm"] == (72,) and t["loop.in"] == (72, 144)
    assert all(t[f"l0.{n}"] == (72,) for n in ("norm1", "norm1b", "norm2", "norm2b"))
    assert t["l0.mix.dq"] == (28, 72) and t["l0.mix.dq.norm"] == (28,) and t["l0.mix.uq"] == (60, 28)
    assert t["l0.mix.dkv"] == (40, 72) and t["l0.mix.dkv.norm"] == (40,) and t["l0.mix.uk"] == (60, 40)
    assert t["l0.mix.uv"] == (100, 40) and t["l0.mix.o"] == (72, 100)
    assert t["l0.mlp.router"] == (9, 72) and t["l0.mlp.correction"] == (9,) and t["l0.mlp.e6.up"] == (24, 72)
    assert "l0.mlp.e7.up" not in t                                       # identity experts have no tensors
    assert t["l0.mlp.shared.gate"] == (48, 72) and t["l0.mlp.shared.down"] == (72, 48) and t["l0.mlp.shared.sg"] == (1, 72)
    assert t["l1.mix.q"] == (120, 72) and t["l1.mix.k"] == (40, 72) and "l1.mix.v" not in t and t["l1.mix.o"] == (72, 120)
    assert t["l1.mlp.up"] == (88, 72) and t["l1.mlp.down"] == (72, 88) and "l1.mlp.gate" not in t
    assert "l2.norm2" not in t and "l4.mlp.shared.sg" not in t and t["l4.mlp.router"] == (6, 72)
    assert "loop.in" not in {s.name for s in DecoderModel(_spec(CONFIG_D)[2]).tensor_specs()}


def test_every_pass_of_the_loop_has_a_cache_and_begins_with_a_join():
    from transformers_neuronx_b200.cache.manager import PagedKVNeed
    from transformers_neuronx_b200.models.decoder import DecoderModel
    _, cfg, spec = _spec(CONFIG_A)
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 1, 2, 1, 2, 3, 4] and [e.cache for e in spec.schedule] == list(range(9))
    assert [e.join is not None for e in spec.schedule] == [False, True, False, True, False, True, False, False, False]
    model = DecoderModel(spec)
    assert len(model.joins) == 1                                         # one set of weights for every pass
    needs = model.cache_needs()
    assert needs[0] == PagedKVNeed(1, 48) and needs[1] == needs[3] == PagedKVNeed(2, 32) and needs[2] == PagedKVNeed(1, 32)
    assert [e.join is not None for e in _spec(CONFIG_B)[2].schedule] == [True, False, False, False] * 2
    assert [e.join is not None for e in _spec(CONFIG_C)[2].schedule] == [False, True, False, False]
    assert not any(e.join for e in _spec(CONFIG_D)[2].schedule)
    d = copy.deepcopy(CONFIG_A)
    d["loop"].pop("start")                                               # absent: from the first layer
    assert _spec(d)[1].layer_runs()[:4] == [(0, True), (1, False), (2, False), (0, True)]


def test_how_the_feed_forwards_are_built():
    from transformers_neuronx_b200.parts import build_part
    _, _, spec = _spec(CONFIG_B)
    ff = [build_part("feed_forward", l.feed_forward) for l in spec.layers]
    assert ff[0].folded and ff[0].always == 1 and ff[0].n_outputs == 16
    assert not ff[1].folded and ff[1].always == 0                        # 160 is no multiple of 96
    assert ff[2].spec.activation == "relu2"
    assert ff[3].folded and ff[3].always == 4
    s = spec.layers[0].feed_forward
    assert (s.n_groups, s.keep_groups, s.group_top, s.scores, s.renormalize) == (4, 2, 1, "softmax", False)
    assert spec.layers[0].mixer.sink == 0.0 and spec.layers[0].mixer.v is None


@pytest.mark.parametrize("edit, word", [
    (lambda d: d["layers"][0].update(type="attention2"), "unknown layer type"),
    (lambda d: d["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda d: d["layers"][0]["mixer"].update(kv_rank=0), "kv_rank"),
    (lambda d: d["layers"][0]["mixer"].update(scale=0.0), "scale"),
    (lambda d: d["layers"][1]["mixer"].update(kv_heads=4), "cannot share"),
    (lambda d: d["layers"][1]["mixer"].update(vdim=24), "vdim must equal dim"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=22), "do not fit"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=7), "do not fit"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(base=-1), "base"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), "not a choice"),       # two groups of three are open
    (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=4), "equal groups"),
    (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "equal groups"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda d: d["layers"][0]["mlp"].update(shared={}), "ff"),
    (lambda d: d["layers"][0]["mlp"].update(kind="gated"), "kind"),
    (lambda d: d["loop"].update(start=3), "not a run"),
    (lambda d: d["loop"].update(stop=6), "not a run"),
    (lambda d: d["loop"].update(times=0), "times"),
    (lambda d: d["norm"].update(eps=0.0), "eps"),
    (lambda d: d.pop("layers"), "layers"),
])
def test_a_configuration_that_cannot_be_is_named(edit, word):
    from transformers_neuronx_b200.config import ConfigError, config_from_dict
    d = copy.deepcopy(CONFIG_A)
    edit(d)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(d)


def test_parts_refuse_what_they_cannot_do():
    import dataclasses
    from transformers_neuronx_b200.models.decoder import DecoderModel
    from transformers_neuronx_b200.models.taborax import _feed_forward
    from transformers_neuronx_b200.parts import build_part
    from transformers_neuronx_b200.parts.spec import LinearSpec, StreamJoinSpec
    spec = _spec(CONFIG_A)[2]
    ff = _feed_forward("m", 72, moe(7, 3, 24, 2, (3, 2), 48))
    for change in (dict(n_identity=3), dict(keep_groups=0), dict(shared=None), dict(n_identity=-1), dict(top=0)):
        with pytest.raises(ValueError):
            build_part("feed_forward", dataclasses.replace(ff, **change))
    with pytest.raises(ValueError):
        build_part("mixer", dataclasses.replace(spec.layers[1].mixer, sink=math.inf))
    for lin in (LinearSpec(72, 72, "w"), LinearSpec(144, 72, "w", "b"), LinearSpec(128, 64, "w")):
        bad = dataclasses.replace(spec, schedule=(dataclasses.replace(spec.schedule[0], join=StreamJoinSpec(lin)),))
        with pytest.raises(ValueError):
            DecoderModel(bad)


def test_a_model_folder_without_the_joins_matrix_is_refused():
    from transformers_neuronx_b200.models.decoder import DecoderModel
    from transformers_neuronx_b200.weights import load_tensors, save_safetensors
    m = TaboraxModel(CONFIG_A, seed=3)
    t = {k: v for k, v in m.plain_tensors.items() if k != "loop.in"}
    save_safetensors(t, m.folder + "/model.safetensors")
    with pytest.raises(Exception, match="loop.in"):
        load_tensors(m.folder, DecoderModel(_spec(CONFIG_A)[2]).tensor_specs())


# ---- the plain implementation's mechanisms ---------------------------------------------------------------
def test_plain_sink_takes_weight_and_gives_no_value():
    s = torch.tensor([[0.0, 9.9], [math.log(3.0), 0.0]], dtype=torch.float64)
    p = BP.softmax_with_sink(s)
    assert torch.allclose(p, torch.tensor([[0.5, 0.0], [0.6, 0.2]], dtype=torch.float64))
    assert torch.allclose(BP.softmax_with_sink(s, math.log(2.0))[0], torch.tensor([1 / 3, 0.0], dtype=torch.float64))


def test_plain_turn_keeps_the_rest_and_depends_on_the_distance_only():
    g = torch.Generator().manual_seed(0)
    q, k = torch.randn(1, 1, 10, generator=g, dtype=torch.float64), torch.randn(1, 1, 10, generator=g, dtype=torch.float64)
    a, b = BP.turn(q.repeat(9, 1, 1), 6, 50.0), BP.turn(k.repeat(9, 1, 1), 6, 50.0)
    assert torch.equal(a[:, :, 6:], q.repeat(9, 1, 1)[:, :, 6:])
    assert abs(float((a[7, 0] * b[3, 0]).sum() - (a[4, 0] * b[0, 0]).sum())) < 1e-6
    assert torch.allclose(a[1, 0, 0], q[0, 0, 0] * math.cos(1.0) - q[0, 0, 3] * math.sin(1.0))


def test_plain_choice_by_corrected_scores_in_the_best_groups():
    s = [0.3, 0.1, 0.25, 0.05, 0.2, 0.1]
    assert BP.choose(s, None, 2) == [0, 2]
    assert BP.choose(s, [0, 0.3, 0, 0, 0, 0], 2) == [1, 0]
    assert BP.choose(s, None, 2, {"count": 3, "keep": 2}) == [0, 2]
    # groups of two: their best are 0.3, 0.25, 0.9; the sum of their two best would have kept the middle one
    assert BP.choose(s, [0, 0, 0, 0, 0.7, -0.9], 3, {"count": 3, "keep": 2}) == [4, 0, 1]
    # negative choice scores stay candidates: the closed groups' experts never come in before them
    assert BP.choose(s, [-1.0, -1.0, -2, -2, -2, -2], 2, {"count": 3, "keep": 1}) == [0, 1]


def test_plain_identity_experts_and_the_gate():
    g = torch.Generator().manual_seed(1)
    rnd = lambda *n: torch.randn(*n, generator=g, dtype=torch.float64)
    h, z = rnd(3, 4), torch.zeros(2, 4, dtype=torch.float64)
    t = {"router": rnd(3, 4), "correction": torch.tensor([0.0, 5.0, 9.0], dtype=torch.float64), "e0.gate": z, "e0.up": z, "e0.down": z.T,
         "shared.gate": rnd(2, 4), "shared.up": rnd(2, 4), "shared.down": rnd(4, 2), "shared.sg": rnd(1, 4)}
    mlp = moe(1, 2, 2, 2, None, 2)
    s = torch.softmax(h @ t["router"].T, -1)
    want = (s[:, 1] + s[:, 2])[:, None] * h + torch.sigmoid(h @ t["shared.sg"].T) * BP.gated(h, t, "shared.")
    assert torch.allclose(BP.experts(h, t, "", mlp), want)


def test_a_wrong_mechanism_would_show():
    """The mechanisms the GPU tests hold the engine to do decide the logits: one of them changed moves the plain logits by
    far more than any tolerance."""
    m = TaboraxModel(CONFIG_A, seed=5)
    ids = m.random_ids(40, 1)
    base = m.plain_logits(ids)

    def moved(edit_cfg=None, edit_t=None, sink=None):
        d, t = copy.deepcopy(m.cfg_dict), dict(m.plain_tensors)
        if edit_cfg:
            edit_cfg(d)
        if edit_t:
            edit_t(t)
        keep, BP.softmax_with_sink = BP.softmax_with_sink, (lambda s: keep(s, sink)) if sink is not None else BP.softmax_with_sink
        try:
            return float((BP.forward_logits(ids, t, d).float() - base).abs().max() / base.abs().max())
        finally:
            BP.softmax_with_sink = keep
    half = lambda t: t.update({"loop.in": torch.cat([t["loop.in"][:, :72], t["loop.in"][:, 72:] * 0], 1)})
    assert moved() == 0.0
    assert moved(sink=-60.0) > 1e-2                                      # no sink
    assert moved(edit_t=half) > 1e-2                                     # the embedding output left out of the join
    assert moved(lambda d: d["loop"].update(times=2)) > 1e-2
    assert moved(lambda d: d["layers"][0]["mlp"]["router"].pop("groups")) > 1e-2
    assert moved(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=1)) > 1e-2
    assert moved(edit_t=lambda t: t.update({"l0.mlp.correction": t["l0.mlp.correction"] * 0})) > 1e-2
    assert moved(edit_t=lambda t: t.update({"l0.mlp.shared.sg": t["l0.mlp.shared.sg"] * 0})) > 1e-3
    assert moved(edit_t=lambda t: t.update({"l0.mix.dq.norm": t["l0.mix.dq.norm"] * 0 + 1})) > 1e-3
    assert moved(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=10)) > 1e-2
