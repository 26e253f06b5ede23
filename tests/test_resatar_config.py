"""The Resatar configuration, its tensors, its caches, the pages that a window with kept first tokens gives back, and the
plain implementation's own mechanisms, without a GPU."""
import copy
import math

import pytest
import torch

from plain import resatar_plain as RP
from resatar_helpers import CONFIG_A, CONFIG_B, CONFIG_C, CONFIGS


def _spec(d):
    from transformers_neuronx_b200.config import config_from_dict
    arch, cfg = config_from_dict(copy.deepcopy(d))
    return arch, cfg, arch.build_spec(cfg)


def test_the_architecture_is_found_by_its_single_name_and_round_trips():
    from transformers_neuronx_b200.config import ResatarConfig, config_from_dict
    for d in CONFIGS.values():
        arch, cfg, spec = _spec(d)
        assert arch.name == "Resatar" and isinstance(cfg, ResatarConfig)
        again = config_from_dict(cfg.to_dict())[1]
        assert again == cfg and again.to_dict()["layers"] == cfg.to_dict()["layers"]
        assert spec.vocab_size == d["vocab"] and spec.hidden_size == d["width"] and len(spec.layers) == len(d["layers"])
        for l in spec.layers:
            assert l.block == "sandwich_norm"
            for n in (l.norm1, l.norm1_post, l.norm2, l.norm2_post):
                assert n is None or (n.one_number and n.eps == d["norm"]["eps"] and n.weight_offset == 0.0)


def test_tensor_names_and_shapes_follow_the_layers():
    from transformers_neuronx_b200.models.decoder import DecoderModel
    _, _, spec = _spec(CONFIG_A)
    t = {s.name: tuple(s.shape) for s in DecoderModel(spec).tensor_specs()}
    assert t["embed"] == (211, 72) and t["head"] == (211, 72) and t["final.norm"] == ()
    assert all(t[f"l0.{n}"] == () for n in ("norm1", "norm1b", "norm2", "norm2b"))
    assert t["l0.mix.q"] == (120, 72) and t["l0.mix.k"] == (40, 72) and t["l0.mix.v"] == (56, 72) and "l0.mix.q.b" not in t
    assert t["l0.mix.g"] == (6, 72) and t["l0.mix.o"] == (72, 168) and t["l0.mix.vmix"] == () and "l3.mix.vmix" not in t
    assert t["l0.mlp.router"] == (6, 72) and t["l0.mlp.router.b"] == (6,) and t["l0.mlp.shared.up"] == (28, 72)
    assert all(t[f"l0.mlp.e{j}.gate"] == (20, 72) and t[f"l0.mlp.e{j}.down"] == (72, 20) for j in range(6)) and "l0.mlp.e6.up" not in t
    assert t["l1.mix.in"] == (120, 72) and t["l1.mix.conv"] == (60, 5) and t["l1.mix.conv.b"] == (60,)
    assert t["l1.mix.x"] == (5 + 36, 60) and t["l1.mix.dt"] == (60, 5) and t["l1.mix.dt.b"] == (60,) and t["l1.mix.o"] == (72, 60)
    assert t["l1.mix.A_log"] == (60, 18) and t["l1.mix.D"] == (60,) and "l1.norm2" not in t and "l1.norm2b" not in t
    p = "l2.mix.left."
    assert t[p + "q"] == (72, 72) and t[p + "q.b"] == (72,) == t[p + "q.norm"] and t[p + "k"] == (36, 72) and t[p + "k.norm"] == (36,)
    assert t[p + "v"] == (60, 72) and t[p + "v.b"] == (60,) and t[p + "g"] == (120, 72) and t[p + "o"] == (72, 120)
    assert t[p + "o.b"] == (72,) and t[p + "r1"] == (6,) == t[p + "r2"] and p + "g.b" not in t
    p = "l2.mix.right."
    assert t[p + "q"] == (90, 72) == t[p + "k"] and t[p + "v"] == (50, 72) == t[p + "g"] and t[p + "o"] == (72, 50) and t[p + "norm"] == (50,)
    assert t["l2.mlp.up"] == (88, 72) and t["l2.mlp.down"] == (72, 88) and "l2.mlp.gate" not in t and "l4.mlp.shared.up" not in t


def test_pages_and_state_of_every_layer():
    from transformers_neuronx_b200.cache.manager import FixedStateNeed, PagedKVNeed, group_needs
    from transformers_neuronx_b200.models.decoder import DecoderModel
    _, _, spec = _spec(CONFIG_A)
    needs = DecoderModel(spec).cache_needs()
    assert needs[0] == PagedKVNeed(2, 32) and needs[3] == PagedKVNeed(3, 32)
    assert needs[(1, 0)] == FixedStateNeed((60, 18), "float32") and needs[(1, 1)] == FixedStateNeed((4, 60), "activation")
    assert needs[(2, 0)] == PagedKVNeed(3, 32, 23, keep_first=5) and needs[(2, 1)] == FixedStateNeed((5, 10, 18), "float32")
    assert needs[(5, 0)] == PagedKVNeed(2, 32)
    groups = group_needs(needs)
    paged = {g.key: (g.window, g.keep_first, g.releases) for g in groups if g.paged}
    assert paged == {("paged", None): (None, 0, False), ("paged", 23, None, 5): (23, 5, True)}
    needs_c = DecoderModel(_spec(CONFIG_C)[2]).cache_needs()
    assert (1, 1) not in needs_c and needs_c[(1, 0)] == FixedStateNeed((50, 70), "float32")      # one tap: no past
    assert needs_c[(4, 0)] == PagedKVNeed(2, 16, 1) and needs_c[(0, 0)] == PagedKVNeed(1, 64, 16, keep_first=17)


@pytest.mark.parametrize("window, keep", [(23, 5), (16, 16), (40, 33), (1, 1), (100, 7)])
def test_the_pages_of_the_first_tokens_stay_and_those_between_are_given_back(window, keep):
    from transformers_neuronx_b200.cache.manager import CacheManager, PagedKVNeed, group_needs
    groups = group_needs({0: PagedKVNeed(1, 16, window, keep_first=keep)})
    m = CacheManager(groups, page_size=16, num_pages=40, max_slots=2)
    m.add_request("a")
    for n in (3, 60, 1, 1, 100, 17, 1, 200):
        m.append("a", n)
        m.release_behind_window("a")
        m.check()
        L, table = m.length("a"), m.block_table("a")
        for pos in range(L):
            needed = pos < keep or pos > L - window                 # some query at position >= L still reads it
            if needed:
                assert table[pos // 16] >= 0, (L, pos)
        held = {b for b, p in enumerate(table) if p >= 0}
        assert held <= {b for b in range(len(table)) if 16 * b < keep or 16 * b + 15 > L - window}
    m.free_request("a")
    m.check()
    assert m.pools[0].num_free == 40


def test_the_values_that_are_mixed_in_come_from_the_first_such_layer():
    _, cfg, spec = _spec(CONFIG_A)
    assert cfg.first_mixing_layer == 0
    assert [getattr(l.mixer, "value_source", "-") for l in spec.layers] == [None, "-", "-", None, 0, "-", 0]
    assert [getattr(l.mixer, "value_mix", "-") for l in spec.layers] == ["l0.mix.vmix", "-", "-", None, "l4.mix.vmix", "-", "l6.mix.vmix"]
    assert _spec(CONFIG_B)[2].layers[3].mixer.value_source == 1


@pytest.mark.parametrize("edit, word", [
    (lambda d: d["layers"][0].update(type="mamba2"), "unknown layer type"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=4), "cannot share"),
    (lambda d: d["layers"][0]["mixer"].update(scale=0.0), "scale"),
    (lambda d: d["layers"][0]["mixer"].update(v_mix=1), "v_mix"),
    (lambda d: d["layers"][4]["mixer"].update(vdim=24), "differs"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=22), "do not fit"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "do not fit"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("low"), "low"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(high=1.0), "exceed"),
    (lambda d: d["layers"][1]["mixer"].pop("dt_rank"), "dt_rank"),
    (lambda d: d["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda d: d["layers"][2]["mixer"].pop("right"), "right"),
    (lambda d: d["layers"][2]["mixer"].pop("left_scale"), "left_scale"),
    (lambda d: d["layers"][2]["mixer"]["right"]["decay"].pop(), "one number for each"),
    (lambda d: d["layers"][2]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][2]["mixer"]["left"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), "not a choice"),
    (lambda d: d["layers"][0]["mlp"].update(shared={}), "ff"),
    (lambda d: d["layers"][2]["mlp"].update(kind="gated"), "kind"),
    (lambda d: d["norm"].update(eps=0.0), "eps"),
    (lambda d: d.pop("layers"), "layers"),
])
def test_a_configuration_that_cannot_be_is_named(edit, word):
    from transformers_neuronx_b200.config import ConfigError, config_from_dict
    d = copy.deepcopy(CONFIG_A)
    edit(d)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(d)


def test_absent_keys_mean_the_mechanism_is_absent():
    d = copy.deepcopy(CONFIG_A)
    m = d["layers"][0]["mixer"]
    for k in ("rot", "v_mix", "kv_heads"):
        m.pop(k)
    d["layers"][2]["mixer"]["left"]["mask"].pop("keep_first")
    _, cfg, spec = _spec(d)
    a = spec.layers[0].mixer
    assert a.rotary is None and a.value_mix is None and a.n_kv_heads == a.n_heads == 6
    assert spec.layers[2].mixer.branches[0].keep_first == 0 and spec.layers[2].mixer.branches[0].window == 23
    assert cfg.first_mixing_layer == 4


@pytest.mark.parametrize("dims, base, scaling", [(64, 1e5, (4.0, 1.0, 4.0, 128)), (20, 2e3, (3.0, 1.0, 2.0, 40)), (12, 1e4, (8.0, 1.5, 6.0, 64)),
                                                (96, 5e5, (16.0, 2.0, 3.0, 1000)), (16, 500.0, None), (2, 10.0, (2.0, 0.01, 0.02, 1.0))])
def test_stretched_frequencies(dims, base, scaling):
    """All three bands occur in the larger cases: kept, blended and slowed."""
    from transformers_neuronx_b200.parts.rotary import inverse_frequencies, rotation_magnitude
    from transformers_neuronx_b200.parts.spec import FrequencyBandsSpec
    sc = dict(zip(("factor", "low", "high", "original"), scaling)) if scaling else None
    got = inverse_frequencies(dims, base, "cpu", FrequencyBandsSpec(**sc) if sc else None)
    want = RP.frequencies(dims, base, sc)
    assert got.dtype == torch.float32 and torch.allclose(got.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-7, atol=0.0)
    plain = RP.frequencies(dims, base)
    if dims >= 64:
        ratio = [w / p for w, p in zip(want, plain)]
        assert any(r == 1.0 for r in ratio) and any(abs(r - 1 / scaling[0]) < 1e-12 for r in ratio)
        assert any(1 / scaling[0] + 1e-6 < r < 1 - 1e-6 for r in ratio)
    assert rotation_magnitude(FrequencyBandsSpec(**sc) if sc else None) == 1.0


# ---- the plain implementation's own mechanisms -------------------------------------------------------
def test_plain_window_and_kept_tokens():
    see = RP.mask(30, 7, 3)
    for i in range(30):
        assert see[i].nonzero().flatten().tolist() == [j for j in range(i + 1) if i - j < 7 or j < 3]
    assert torch.equal(RP.mask(9), torch.tril(torch.ones(9, 9, dtype=torch.bool)))


def test_plain_distance_bias_is_a_power_of_the_distance():
    """With equal scores the weights are (1 + r2 d)^(-r1)."""
    T, r1, r2 = 12, 1.5, 0.4
    v = torch.eye(T, dtype=torch.float64).reshape(T, 1, T)
    o = RP.attend(torch.zeros(T, 1, 4, dtype=torch.float64), torch.zeros(T, 1, 4, dtype=torch.float64), v, 1.0, RP.mask(T),
                  lambda h: RP.distance_bias(T, r1, r2))[:, 0]
    w = torch.tensor([(1 + r2 * d) ** -r1 for d in range(T)], dtype=torch.float64)
    for i in range(T):
        assert torch.allclose(o[i, :i + 1], w[:i + 1].flip(0) / w[:i + 1].sum(), atol=1e-12)


def test_plain_scan_and_lightning_as_sums_over_the_past():
    g = torch.Generator().manual_seed(0)
    T, C, N = 9, 3, 4
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    x, dt, A, B, Cm, D = rnd(T, C), rnd(T, C).abs(), -rnd(C, N).abs(), rnd(T, N), rnd(T, N), rnd(C)
    y, _ = RP.scan(x, dt, A, B, Cm, D)
    for t in range(T):
        for c in range(C):
            want = D[c] * x[t, c]
            for s in range(t + 1):
                want = want + (torch.exp(A[c] * dt[s + 1:t + 1, c].sum()) * dt[s, c] * x[s, c] * B[s] * Cm[t]).sum()
            assert abs(float(y[t, c] - want)) < 1e-10
    m = {"heads": 1, "dim": 3, "vdim": 2, "decay": [0.8]}
    t = {"q": rnd(3, 5), "k": rnd(3, 5), "v": rnd(2, 5), "g": torch.zeros(2, 5, dtype=torch.float64), "norm": torch.ones(2, dtype=torch.float64),
         "o": torch.eye(2, dtype=torch.float64)}
    h = rnd(T, 5)
    got = RP.lightning(h, t, "", m, 1e-12)
    q, k, v = (RP.silu(h @ t[n].T) for n in "qkv")
    for i in range(T):
        o = sum(0.8 ** (i - j) * float(q[i] @ k[j]) * v[j] for j in range(i + 1))
        assert torch.allclose(got[i], 0.5 * o / math.sqrt(float((o * o).mean())), atol=1e-9)


def test_plain_routing_is_a_softmax_over_the_chosen_logits():
    h = torch.eye(4, dtype=torch.float64)
    t = {"router": torch.tensor([[1.0, 0, 0, 0], [0, 2.0, 0, 0], [0, 0, 3.0, 0]], dtype=torch.float64), "router.b": torch.tensor([0.0, 0.5, -4.0], dtype=torch.float64)}
    picks = RP.route(h, t, "", 2)
    assert [p[0] for p in picks] == [[0, 1], [1, 0], [1, 0], [1, 0]]
    assert abs(float(picks[1][1][0]) - 1 / (1 + math.exp(-2.5))) < 1e-12


def test_a_wrong_window_sink_or_bias_would_show():
    """The mechanisms the GPU tests hold the engine to do decide the logits: with the window one wider or narrower, one first
    token more or fewer, the bias left out, or the values not mixed, the plain logits move by far more than any tolerance."""
    from resatar_helpers import ResatarModel
    m = ResatarModel(CONFIG_A, seed=5)
    ids = m.random_ids(60, 1)
    base = m.plain_logits(ids)

    def moved(edit_cfg=None, edit_t=None):
        d, t = copy.deepcopy(m.cfg_dict), dict(m.plain_tensors)
        if edit_cfg:
            edit_cfg(d)
        if edit_t:
            edit_t(t)
        return float((RP.forward(d, t, ids).float() - base).abs().max() / base.abs().max())
    mask = lambda d: d["layers"][2]["mixer"]["left"]["mask"]
    assert moved(lambda d: mask(d).update(size=24)) > 1e-3 and moved(lambda d: mask(d).update(size=22)) > 1e-3
    assert moved(lambda d: mask(d).update(keep_first=6)) > 1e-3 and moved(lambda d: mask(d).update(keep_first=4)) > 1e-3
    assert moved(edit_t=lambda t: t.update({"l2.mix.left.r1": t["l2.mix.left.r1"] * 0})) > 1e-3
    assert moved(edit_t=lambda t: t.update({"l4.mix.vmix": t["l4.mix.vmix"] * 0})) > 1e-3
    assert moved(edit_t=lambda t: t.update({"l0.mix.vmix": t["l0.mix.vmix"] + 5.0})) == 0.0       # the first layer's is unused
    assert moved(edit_t=lambda t: t.update({"l0.mlp.router.b": t["l0.mlp.router.b"] * 0})) > 1e-3
    assert moved(lambda d: d["layers"][0]["mixer"]["rot"].pop("scaling")) > 1e-3
