"""The Taborax decoder on the GPU against the plain implementation (tests/plain/taborax_plain.py): every mechanism's kernel
alone, then whole models through the replay program's function (whole prompts, token by token, portions down to two
tokens, mixed batches with pages used again), far keys and a sink made to decide, long decoding, and greedy generation
through the engine's own entry point and scheduler."""
import dataclasses
import math

import pytest
import torch

from helpers import run_trace_inprocess
from plain import taborax_plain as BP
from taborax_helpers import (CONFIG_A, CONFIGS, TOLERANCE, TaboraxModel, attn, compare, cut_steps, dense, latent, layer,
                             mixed_steps, moe, whole_steps)

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64
_models = {}


def _decided(t):
    """Corrections eight times as far apart, so that hardly a token's choice of experts is a close call."""
    for name in t:
        if name.endswith(".correction"):
            t[name] = t[name] * 8


def _model(name, dtype="float32"):
    """B in bfloat16 has decided choices: with the weights as drawn, rounding the inputs of the plain implementation's products
    to bfloat16 changes one choice in fifty (each changes its row, and every later one a little), which is all one would see."""
    key = (name, dtype if name == "B" else None)
    if key not in _models:
        _models[key] = TaboraxModel(CONFIGS[name], seed=5, edit=_decided if key[1] == "bfloat16" else None)
    return _models[key]


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def _close(got, want, tol):
    err = float((got.double().cpu() - want.double()).abs().max()) / max(float(want.abs().max()), 1e-30)
    assert err <= tol, err


def _step_context(N, dtype, pad=0):
    from transformers_neuronx_b200.parts.base import StepContext
    ctx = StepContext(torch.device(DEV), dtype)
    ctx.n_tokens = N + pad
    ctx.token_request = _i32([0] * N + [-1] * pad)
    return ctx


# ---- the sink in every attention kernel ---------------------------------------------------------------
def _plain_rows(q, k, v, scale, sink, window, rows, bias=None):
    """Rows of softmax(scores) v with one more key of score `sink` and without a value."""
    L, H, D = q.shape
    G = k.shape[1]
    i, j = torch.arange(L)[:, None], torch.arange(L)[None, :]
    out = torch.zeros(L, H, D, dtype=F64)
    for h in range(H):
        s = (q[:, h].double() @ k[:, h // (H // G)].double().T) * scale
        if bias is not None:
            s = s - bias[0][h].double() * torch.log(1 + bias[1][h].double() * (i - j).clamp(min=0))
        if window:
            s = s.masked_fill(i - j >= window, -math.inf)
        out[:, h] = BP.softmax_with_sink(s, sink) @ v[:, h // (H // G)].double()
    return out[rows].reshape(len(rows), -1)


@pytest.mark.parametrize("H, G, D, dtype", [(4, 2, 32, torch.float32), (6, 3, 48, torch.bfloat16), (4, 1, 96, torch.bfloat16),
                                            (8, 2, 128, torch.bfloat16), (2, 2, 64, torch.bfloat16), (2, 1, 160, torch.bfloat16),
                                            (3, 1, 272, torch.bfloat16)])
@pytest.mark.parametrize("sink, shift, window, biased", [(0.0, 0.0, 0, False), (0.0, -7.0, 0, False), (0.0, 20.0, 0, False),
                                                         (2.5, 0.0, 37, False), (-3.0, -5.0, 1, True), (9.0, 3.0, 64, True)])
def test_a_sink_in_prompts_and_decoding(H, G, D, dtype, sink, shift, window, biased):
    """A context of 301 positions on shuffled pages: its last 201 rows as one portion, its first 40 as another, single rows
    as decode rows with their own key appended by the kernel, under several splits of the context.  `shift` moves all of
    a head's scores: far below the sink it takes nearly all the weight, far above it next to none."""
    from transformers_neuronx_b200.kernels import ops
    g = torch.Generator().manual_seed(11)
    L, scale = 301, 0.17
    f = (3.0 / (scale * D ** 0.5)) ** 0.5
    q, k, v = torch.randn(L, H, D, generator=g) * f, torch.randn(L, G, D, generator=g) * f, torch.randn(L, G, D, generator=g)
    q[:, :, 0], k[:, :, 0] = math.copysign(1.0, shift) * (abs(shift) / scale) ** 0.5, (abs(shift) / scale) ** 0.5
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    bias = (torch.rand(H, generator=g), torch.rand(H, generator=g)) if biased else None
    blocks = -(-L // 16)
    pages = torch.randperm(blocks + 3, generator=g)[:blocks].tolist()
    cache = torch.randn(blocks + 3, 2, G, 16, D, generator=g).to(dtype)
    for b in range(blocks):
        n = min(16, L - 16 * b)
        cache[pages[b], 0, :, :n] = k[16 * b:16 * b + n].transpose(0, 1)
        cache[pages[b], 1, :, :n] = v[16 * b:16 * b + n].transpose(0, 1)
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    dev, bt = cache.to(DEV), _i32([pages])
    kw = dict(window=window, sink=sink, bias=None if bias is None else (bias[0].to(DEV), bias[1].to(DEV)))
    for first, n in ((L - 201, 201), (0, 40)):
        rows = list(range(first, first + n))
        want = _plain_rows(q, k, v, scale, sink, window, rows, bias)
        qs = q[rows].reshape(n, H * D).contiguous().to(DEV)
        out = torch.empty_like(qs)
        ops.attention_simt(qs, dev, bt, _i32([0] * n), _i32(rows), out, H, scale, **kw)
        _close(out, want, tol)
        if dtype == torch.float32 or D > 256:
            continue
        tiles = list(range(0, n, 128))
        args = (qs, dev, bt, _i32([0] * len(tiles)), _i32(tiles), _i32([0]), _i32([n]), _i32([first]), out, H, scale)
        out.zero_()
        ops.attention_prefill(*args, **kw)
        _close(out, want, tol)
        if ops.attention_prefill_tc_supported(qs, dev, out):
            out.zero_()
            ops.attention_prefill_tc(*args, **kw)
            _close(out, want, tol)
    if dtype == torch.float32 or D > 256:
        return
    ps = [0, 1, 14, 15, 16, 17, 63, 64, 200, L - 1]
    want = _plain_rows(q, k, v, scale, sink, window, ps, bias)
    bt = _i32([pages] * len(ps))
    qs = q[ps].reshape(len(ps), H * D).contiguous().to(DEV)
    kn, vn = k[ps].reshape(len(ps), G * D).contiguous().to(DEV), v[ps].reshape(len(ps), G * D).contiguous().to(DEV)
    for plan in (dict(), dict(n_splits=1, warps=4), dict(n_splits=3, warps=4), dict(n_splits=7, warps=8), dict(grouped=True), dict(grouped=False)):
        for new in ((kn, vn), None):
            out = torch.empty(len(ps), H * D, device=DEV, dtype=dtype)
            ops.attention_decode(qs, dev, bt, _i32(list(range(len(ps)))), _i32(ps), out, H, scale, max_kv_len=L, new_kv=new, **kw, **plan)
            _close(out, want, tol)


# ---- the feed-forwards ---------------------------------------------------------------------------------
@pytest.mark.parametrize("E, identity, top, groups, always, gated, W", [
    (7, 2, 3, (3, 2), 2, True, 72), (16, 0, 4, None, 0, True, 256), (1, 1, 1, None, 1, True, 33), (60, 4, 8, (8, 3), 4, True, 128),
    (3, 3, 2, (6, 4), 0, False, 50), (5, 1, 6, None, 1, False, 64), (100, 30, 2, (2, 1), 0, False, 64)])
def test_routing(E, identity, top, groups, always, gated, W):
    """Choice by softmax score plus correction in the groups with the best single experts, weights that are the scores alone,
    identity experts marked -2, the experts that every token takes behind the chosen ones with the gate as weight."""
    from transformers_neuronx_b200.kernels import ops
    g = torch.Generator().manual_seed(7)
    N, R = 40, E + identity
    h, router = torch.randn(N, W, generator=g), torch.randn(R, W, generator=g) * 2 * W ** -0.5
    sg, corr = torch.randn(1, W, generator=g) * W ** -0.5, torch.randn(R, generator=g) / R
    if R > 4:
        corr[R // 2] = -2.0                                              # choice scores may be negative
    s = torch.softmax(h.double() @ router.double().T, -1)
    gate = torch.sigmoid(h.double() @ sg.double().T)[:, 0]
    ids = torch.empty(N + 1, top + always, dtype=torch.int32, device=DEV)
    wts, go = torch.empty(N + 1, top + always, device=DEV), torch.full((N + 1,), 9.0, device=DEV)
    ops.moe_route(torch.cat([h, torch.zeros(1, W)]).to(DEV), torch.cat([router, sg]).to(DEV) if gated else router.to(DEV),
                  _i32([0] * N + [-1]), ids, wts, top, softmax_scores=True, correction=corr.to(DEV),
                  n_groups=groups[0] if groups else 1, keep_groups=groups[1] if groups else 1, group_top=1, always=always,
                  n_identity=identity, gated=gated, gate_out=go if gated else None)
    assert ids[N].tolist() == [-1] * (top + always)
    seen = set()
    for n in range(N):
        want = BP.choose(s[n], corr, top, {"count": groups[0], "keep": groups[1]} if groups else None)
        seen |= set(want)
        assert ids[n].tolist() == [e if e < E else -2 for e in want] + [E + i for i in range(always)], n
        _close(wts[n, :top], s[n, want], 5e-6)
        _close(wts[n, top:], (gate[n] if gated else torch.ones((), dtype=F64)).expand(always), 5e-6) if always else None
    if identity:
        assert any(e >= E for e in seen) and any(e < E for e in seen)
    if gated:
        _close(go[:N], gate, 5e-6)


EXPERTS = [(7, 3, 24, 2, (3, 2), 48, 72, 5, torch.float32), (7, 3, 24, 2, (3, 2), 48, 72, 200, torch.float32),
           (4, 2, 36, 4, None, 30, 72, 9, torch.float32), (5, 2, 40, 1, None, None, 72, 9, torch.float32),
           (12, 4, 64, 4, (4, 2), 64, 256, 1, torch.bfloat16), (12, 4, 64, 4, (4, 2), 64, 256, 300, torch.bfloat16), (12, 4, 64, 4, (4, 2), 64, 256, 600, torch.bfloat16),
           (6, 2, 32, 2, None, 128, 256, 40, torch.bfloat16), (6, 2, 32, 2, None, 128, 256, 515, torch.bfloat16), (8, 1, 96, 0, (2, 1), 160, 256, 40, torch.bfloat16),
           (1, 1, 20, 1, None, 20, 100, 33, torch.bfloat16), (3, 2, 12, 3, (6, 4), 36, 100, 7, torch.bfloat16),
           (2, 4, 32, 6, None, 32, 64, 50, torch.bfloat16)]


@pytest.mark.parametrize("E, top, ff, identity, groups, shared, W, N, dtype", EXPERTS)
def test_experts_identity_experts_and_a_gated_shared_one(E, top, ff, identity, groups, shared, W, N, dtype, monkeypatch):
    """The shared expert in the experts' products (their width or a multiple) and as a feed-forward of its own, rows all of
    whose choices are identity experts, a padded row; written and added; in one launch and in several."""
    from transformers_neuronx_b200.kernels import ops
    from transformers_neuronx_b200.models.taborax import _feed_forward
    from transformers_neuronx_b200.parts import build_part
    g = torch.Generator().manual_seed(8)
    mlp = moe(E, top, ff, identity, groups, shared)
    part = build_part("feed_forward", _feed_forward("m", W, mlp))
    assert part.folded == (shared is not None and shared % ff == 0)
    t = {s.name: (torch.randn(s.shape, generator=g) * 0.15).to(dtype) for s in part.tensor_specs()}
    t["m.router"] = (t["m.router"].float() * 4).to(dtype)
    part.load(t, torch.device(DEV), dtype)
    h = torch.randn(N, W, generator=g).to(dtype)
    plain = {k[2:]: v.double() for k, v in t.items()}
    want = BP.experts(h.double(), plain, "", mlp)
    hs = torch.cat([h, torch.zeros(1, W, dtype=dtype)]).to(DEV)
    # as many tokens choose it; the few-pairs launches of the 32-bit form; the folded shared expert as dense products
    for most, apart in ((8192, type(part).APART_FROM), (7 * (top + part.always), 1)):
        monkeypatch.setattr(ops, "MOE_PAIRS_PER_LAUNCH", most)
        monkeypatch.setattr(type(part), "APART_FROM", apart)
        ctx = _step_context(N, dtype, pad=1)
        for accumulate in (False, True):
            out = torch.full((N + 1, W), 1.0, device=DEV)
            part.forward(ctx, hs, out, accumulate=accumulate)
            _close(out[:N], want + (1.0 if accumulate else 0.0), 1e-5 if dtype == torch.float32 else 2e-2)
            if shared is None or (part.folded and (apart > N or part.shared_down is None or W % 8 or ff % 8)):
                assert float((out[N] - 1.0).abs().max()) == 0.0           # the padded row is left alone
            ctx.begin_entry()


@pytest.mark.parametrize("N, F, dtype", [(5, 48, torch.float32), (130, 512, torch.bfloat16), (3, 30, torch.bfloat16)])
def test_a_number_per_row_on_the_gated_activation(N, F, dtype):
    from transformers_neuronx_b200.kernels import ops
    g = torch.Generator().manual_seed(9)
    gu, rs = torch.randn(N, 2 * F, generator=g).to(dtype), torch.randn(N, generator=g) * 3
    out = torch.empty(N, F, device=DEV, dtype=dtype)
    ops.gated_activation(gu.to(DEV), out, "silu", rs.to(DEV))
    _close(out, BP.silu(gu[:, :F].double()) * gu[:, F:].double() * rs.double()[:, None], 2e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("N, K, F", [(300, 128, 512), (130, 72, 88), (5, 256, 512), (1, 256, 512), (2048, 64, 1000), (7, 33, 50)])
def test_squared_relu_behind_the_up_product(N, K, F):
    """In the products' epilogues: whole tiles, ragged edges, few tokens, one token, sizes the tensor-core product refuses."""
    from transformers_neuronx_b200.parts.linear import Linear
    from transformers_neuronx_b200.parts.spec import LinearSpec
    g = torch.Generator().manual_seed(9)
    for dtype in (torch.bfloat16, torch.float32):
        lin = Linear(LinearSpec(K, F, "w"))
        w = (torch.randn(F, K, generator=g) * torch.logspace(-2, 0, F)[:, None]).to(dtype)
        lin.load({"w": w}, torch.device(DEV), dtype)
        a = torch.randn(N, K, generator=g).to(dtype)
        out = torch.empty(N, F, device=DEV, dtype=dtype)
        lin.forward(a.to(DEV), out, activation="relu2")
        want = torch.clamp(a.double() @ w.double().T, min=0.0) ** 2
        err = (out.cpu().double() - want).abs()
        assert float((err - (1e-4 if dtype == torch.float32 else 2.0 ** -8) * want).max()) <= 1e-4
        assert bool((out.cpu()[want == 0.0] == 0).all())


# ---- the join of the stream with the embedding output --------------------------------------------------
@pytest.mark.parametrize("N, W, dtype", [(1, 72, torch.float32), (130, 72, torch.float32), (1, 256, torch.bfloat16),
                                         (40, 256, torch.bfloat16), (300, 256, torch.bfloat16), (9, 100, torch.bfloat16)])
def test_a_join_is_one_product_of_both(N, W, dtype):
    from transformers_neuronx_b200.parts import StreamJoin
    from transformers_neuronx_b200.parts.spec import LinearSpec, StreamJoinSpec
    g = torch.Generator().manual_seed(4)
    w = (torch.randn(W, 2 * W, generator=g) * W ** -0.5).to(dtype)
    part = StreamJoin(StreamJoinSpec(LinearSpec(2 * W, W, "w")))
    part.load({"w": w}, torch.device(DEV), dtype)
    x0 = torch.randn(N, W, generator=g).to(dtype)
    ctx = _step_context(N, dtype)
    start = part.begin(ctx, x0.to(DEV))
    for x in (torch.randn(N, W, generator=g) * 5, x0.float(), torch.randn(N, W, generator=g)):     # several passes of a step
        xd = x.to(DEV)
        part.forward(ctx, xd, xd.to(dtype), start)
        _close(xd, torch.cat([x.to(dtype).double(), x0.double()], -1) @ w.double().T, 2e-6 if dtype == torch.float32 else 1e-4)


@pytest.mark.parametrize("block", ["pre_norm", "output_norm", "post_norm"])
def test_joins_ahead_of_blocks_of_other_kinds(block):
    """A join takes the stream as any block leaves it, also one that keeps no copy of it or works on a copy of its own."""
    from transformers_neuronx_b200.config import config_from_dict
    from transformers_neuronx_b200.engine import build_model
    from transformers_neuronx_b200.engine.step import StepEntry, StepRunner
    cfg = {"architecture": "Taborax", "vocab": 97, "width": 48, "norm": {"eps": 1e-5}, "init_std": 0.2,
           "loop": {"start": 0, "stop": 2, "times": 2},
           "layers": [layer(attn(4, 2, 16, 0.3, 8, 100.0), dense(40)), layer(latent(3, 12, 8, 10, 20, 0.3), dense(56))]}
    m = TaboraxModel(cfg, seed=6)
    arch, c = config_from_dict(cfg)
    spec = arch.build_spec(c)
    spec = dataclasses.replace(spec, layers=tuple(dataclasses.replace(l, block=block) for l in spec.layers))
    model = build_model(spec, m.plain_tensors, "float32", verbose=False)
    ids = m.random_ids(37, 2)
    t = {k: v.double() for k, v in m.plain_tensors.items()}
    norm = lambda y, name: BP.rms(y, 1e-5, t[name])
    x0 = x = t["embed"][ids]
    for i, begins in BP.walk(cfg):
        p, l = f"l{i}.", cfg["layers"][i]
        if begins:
            x = torch.cat([x, x0], -1) @ t["loop.in"].T
        mix = (lambda h: BP.sink_attention(h, t, p + "mix.", l["mixer"])) if i == 0 else \
            (lambda h: BP.latent_attention(h, t, p + "mix.", l["mixer"], 1e-5))
        ff = lambda h: BP.dense(h, t, p + "mlp.")
        if block == "pre_norm":
            x = x + mix(norm(x, p + "norm1"))
            x = x + ff(norm(x, p + "norm2"))
        elif block == "output_norm":
            x = x + norm(mix(x), p + "norm1")
            x = x + norm(ff(x), p + "norm2")
        else:
            x = norm(x + mix(x), p + "norm1")
            x = norm(x + ff(x), p + "norm2")
    want = norm(x, "final.norm") @ t["head"].T
    runner = StepRunner(model, page_size=16, num_pages=8, max_slots=2, max_model_len=128, use_cuda_graphs=True)
    runner.add_request("a")
    _close(runner.step([StepEntry("a", ids[:20], list(range(20)))]), want[:20], 5e-5)
    for i in range(20, 37):
        _close(runner.step([StepEntry("a", [ids[i]], [0])]), want[i:i + 1], 5e-5)
    runner.finish("a")


# ---- whole models through the replay function ------------------------------------------------------------
LENGTHS = {"A": [1, 2, 17, 45, 130], "B": [3, 140, 300]}
# The rows' median error in bfloat16: A walks nine layer runs of width 72 and B eight, fifteen sublayers each normalised to
# unit size before it joins the stream, so that each one's rounding arrives in full (measured under every cut alike: 3.5e-2 in
# B).  The 32-bit engine holds every row to 3e-5.
BF16_MEDIAN = {"A": 7e-2, "B": 5e-2, "C": 5e-2, "D": TOLERANCE["bfloat16"]}


def _tol(name, dtype):
    return BF16_MEDIAN[name] if dtype == "bfloat16" else None


def _requests(m, lengths, seed=100):
    return {f"r{i}": m.random_ids(n, seed=seed + i) for i, n in enumerate(lengths)}


@pytest.mark.parametrize("name", ["A", "B"])
def test_the_stream_after_every_layer_run(name):
    """The residual stream after each run of a layer (a looped layer counts every pass) against the plain one: the first
    wrong run names the mechanism."""
    from transformers_neuronx_b200.engine import load_model
    from transformers_neuronx_b200.engine.step import StepEntry, StepRunner
    m = _model(name)
    ids = m.random_ids(70, 11)
    want = m.plain_hidden(ids)                                           # [runs, T, width]
    model, _ = load_model(m.folder, "float32", verbose=False)
    runner = StepRunner(model, page_size=16, num_pages=8, max_slots=2, max_model_len=128, use_cuda_graphs=False)
    runner.add_request("a")
    with model.tap_hidden_states() as taps:
        runner.step([StepEntry("a", ids, [len(ids) - 1])])
        torch.cuda.synchronize()
        assert want.shape[0] == len(model.spec.schedule) and f"entry{want.shape[0]}" not in taps
        for run in range(want.shape[0]):
            _close(taps[f"entry{run}"][:len(ids)], want[run], 2e-5)
    runner.finish("a")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_whole_prompts(name, dtype):
    m = _model(name, dtype)
    reqs = _requests(m, LENGTHS[name])
    steps = whole_steps(reqs)
    compare(m, reqs, steps, run_trace_inprocess(m.folder, dtype, steps, 64 * 5), dtype, tol=_tol(name, dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_a_prefix_then_token_by_token(name, dtype):
    """Decoding through the pages, over several pages' borders; the decode steps are replayed from a captured graph."""
    m = _model(name, dtype)
    reqs = _requests(m, [n for n in LENGTHS[name] if n > 71])
    steps = cut_steps(reqs, [1000], tail=70)
    compare(m, reqs, steps, run_trace_inprocess(m.folder, dtype, steps, 64 * 5), dtype, tol=_tol(name, dtype))


def test_from_the_first_token_on_one_by_one():
    """The first positions, where the sink holds the most weight."""
    m = _model("A")
    reqs = _requests(m, [50])
    steps = cut_steps(reqs, [1])
    compare(m, reqs, steps, run_trace_inprocess(m.folder, "float32", steps, 64), "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_portions_of_changing_size_down_to_two_tokens(name, dtype):
    """Portions that end one before, at and one behind a page's border, pairs, and one longer than a tile of queries."""
    m = _model(name, dtype)
    reqs = _requests(m, LENGTHS[name][-2:])
    steps = cut_steps(reqs, [2, 33, 3, 16, 2, 17, 64, 5, 15, 130], tail=3)
    compare(m, reqs, steps, run_trace_inprocess(m.folder, dtype, steps, 64 * 5), dtype, tol=_tol(name, dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_mixed_batches_with_pages_used_again(name, dtype):
    """More requests than the replay program has slots: a finished request's pages (of every pass of a looped layer) go to
    the next request, and the pool holds no more than the live requests need."""
    m = _model(name, dtype)
    lengths = [90, 7, 33, 150, 12, 64, 5, 49, 2, 120, 31] if name == "A" else [150, 20, 70, 9, 200, 40, 33, 129, 18]
    reqs = _requests(m, lengths, seed=300)
    steps = mixed_steps(reqs, [9, 2, 31, 16, 5, 64, 3])
    most = sorted(-(-n // 64) * 64 for n in lengths)[-4:]
    compare(m, reqs, steps, run_trace_inprocess(m.folder, dtype, steps, sum(most)), dtype, tol=_tol(name, dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["C", "D"])
def test_sizes_that_no_fast_path_takes(name, dtype):
    """C: widths that are no multiples of 8; D: rows of more than 256 dims a position."""
    m = _model(name, dtype)
    reqs = _requests(m, [3, 70, 41], seed=600)
    for steps in (whole_steps(reqs), mixed_steps(reqs, [7, 2, 19, 33], decode_tail=12)):
        compare(m, reqs, steps, run_trace_inprocess(m.folder, dtype, steps, 64 * 4), dtype, tol=_tol(name, dtype))


def test_logits_do_not_depend_on_the_cut_or_the_batch_beyond_rounding():
    m = _model("A")
    reqs = _requests(m, [130, 45], seed=500)
    runs = []
    for steps in (whole_steps(reqs), cut_steps(reqs, [2, 16, 17, 1, 31]), mixed_steps(reqs, [15, 2, 40], decode_tail=20)):
        res = run_trace_inprocess(m.folder, "float32", steps, 64 * 4)
        at, out = {r: 0 for r in reqs}, {}
        for s in steps:
            row = 0
            for e in s["entries"]:
                for w in e["want"]:
                    out[(e["id"], at[e["id"]] + w)] = torch.from_numpy(res[s["step"]][row].copy()); row += 1
                at[e["id"]] += len(e["tokens"])
        runs.append(out)
    for other in runs[1:]:
        for key, lg in other.items():
            assert float((lg - runs[0][key]).abs().max()) <= 2e-5 * float(runs[0][key].abs().max()), key


# ---- single keys and the sink, made to decide --------------------------------------------------------------
def _one(mixer, **more):
    return dict({"architecture": "Taborax", "vocab": 97, "width": 64, "norm": {"eps": 1e-5}, "init_std": 0.3,
                 "layers": [layer(mixer, None)]}, **more)


def _far_steps(reqs):
    return (whole_steps(reqs), cut_steps(reqs, [33, 15, 2, 17, 16, 1, 64], tail=41), mixed_steps(reqs, [31, 2, 48, 17], decode_tail=35))


@pytest.mark.parametrize("loop", [None, {"start": 0, "stop": 1, "times": 2}])
@pytest.mark.parametrize("mixer", [latent(4, 16, 24, 20, 28, 6.0), attn(4, 2, 32, 2.0, 16, 1000.0)])
def test_a_far_key_among_hundreds(mixer, loop):
    """A large scale makes every softmax nearly one-hot: rows that single keys from anywhere in the sequence decide (or the
    sink, where all scores are negative).  A page, a pass' cache, a latent or a rotation that is off picks another value."""
    m = TaboraxModel(_one(mixer, **({"loop": loop} if loop else {})), seed=24)
    reqs = {"a": m.random_ids(300, 1), "b": m.random_ids(61, 2)}
    for steps in _far_steps(reqs):
        compare(m, reqs, steps, run_trace_inprocess(m.folder, "float32", steps, 64 * 6), "float32", tol=3e-4)


def test_a_marked_key_is_found_from_every_distance():
    """Token 7 is the mark and stands once, at position 5.  The rotated dims carry nothing; every token's query and the mark's
    key share a direction that no other key has, so every later row reads the mark's value."""
    cfg = _one(attn(2, 1, 24, 1.0, 8, 100.0), width=64)

    def mark(t):
        e = torch.randn(97, 64, generator=torch.Generator().manual_seed(3)) * 0.5
        e[:, :2] = 0.0
        e[:, 0] = 2.0                                                    # every token's query comes from here
        e[7, 1] = 3.0                                                    # the mark's key from here
        t["embed"] = e.to(torch.bfloat16)
        for name, col in (("q", 0), ("k", 1)):
            w = t[f"l0.mix.{name}"].float() * 0.05
            w.view(-1, 24, 64)[:, :8] = 0.0                              # the rotated dims
            w[:, :2] = 0.0
            w.view(-1, 24, 64)[:, 8:, col] = 2.0
            t[f"l0.mix.{name}"] = w.to(torch.bfloat16)
    m = TaboraxModel(cfg, seed=25, edit=mark)
    ids = [x if x != 7 else 8 for x in m.random_ids(420, 1)]
    ids[5] = 7
    plain = m.plain_logits(ids)
    without = m.plain_logits([8 if x == 7 else x for x in ids])
    assert float((plain[300:] - without[300:]).abs().max(-1).values.min()) > 0.1 * float(plain.abs().max())
    reqs = {"a": ids}
    for steps in (whole_steps(reqs), cut_steps(reqs, [100, 2, 31, 16], tail=200)):
        for dtype in ("float32", "bfloat16"):
            compare(m, reqs, steps, run_trace_inprocess(m.folder, dtype, steps, 64 * 7), dtype)


def test_scores_far_below_the_sink_leave_next_to_nothing():
    """All scores far below 0: the softmax without a sink would be as sharp as ever, with it a row's output shrinks by
    e^score, which the norm behind the mixer (eps inside the root) turns into rows that differ wholesale."""
    cfg = _one(attn(2, 1, 24, 1.0), norm={"eps": 1e-3})

    def low(t):
        t["embed"][:, 0] = 3.0
        for name, sign in (("q", 1.0), ("k", -1.0)):
            w = t[f"l0.mix.{name}"].float() * 0.2
            w[:, 0] = sign * 0.1
            t[f"l0.mix.{name}"] = w.to(torch.bfloat16)
    m = TaboraxModel(cfg, seed=26, edit=low)
    ids = m.random_ids(90, 1)
    keep = BP.softmax_with_sink
    BP.softmax_with_sink = lambda s: keep(s, -80.0)
    try:
        without = BP.forward_logits(ids, m.plain_tensors, m.cfg_dict).float()
    finally:
        BP.softmax_with_sink = keep
    plain = m.plain_logits(ids)
    off = (plain - without).abs().max(-1).values / plain.abs().max()
    assert float(off.median()) > 0.1, off
    reqs = {"a": ids}
    for steps in (whole_steps(reqs), cut_steps(reqs, [2, 31, 16], tail=20)):
        for dtype in ("float32", "bfloat16"):
            compare(m, reqs, steps, run_trace_inprocess(m.folder, dtype, steps, 64 * 2), dtype)


def test_long_decoding():
    m = _model("A")
    reqs = _requests(m, [260], seed=700)
    steps = cut_steps(reqs, [4], tail=250)
    compare(m, reqs, steps, run_trace_inprocess(m.folder, "float32", steps, 64 * 5), "float32")


# ---- the engine's own entry point ------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(dtype):
    from transformers_neuronx_b200.config import EngineConfig
    from transformers_neuronx_b200.engine import LLMEngine, load_model
    m = _model("B", dtype)
    model, typed = load_model(m.folder, dtype, verbose=False)
    eng = LLMEngine(model, EngineConfig(dtype=dtype, max_num_seqs=3, max_batch_tokens=48, max_portion=20, max_tokens=640,
                                        max_model_len=256))
    prompts = [m.random_ids(n, 900 + n) for n in (37, 5, 70, 18)]
    outs = eng.generate(prompts, 12, stop_on_eos=False)
    far = 0
    for prompt, out in zip(prompts, outs):
        assert len(out) == 12
        logits = m.plain_logits(list(prompt) + list(out))
        for i, tok in enumerate(out):
            lg = logits[len(prompt) - 1 + i]
            if tok != int(lg.argmax()):                      # a tie that rounding may decide either way
                far += float(lg.max() - lg[tok]) / float(lg.abs().max()) > 2 * (TOLERANCE[dtype] if dtype == "float32" else BF16_MEDIAN["B"])
    assert far <= (0 if dtype == "float32" else 2)           # in bfloat16 a row whose experts are a close call may differ
    eng.runner.cache.check()
    assert eng.runner.cache.slots.num_free == 3


def test_the_entry_point_class_and_the_command_line(tmp_path):
    """config.json picks the entry-point class; greedy `sample` equals the plain argmax, teacher-forced; the demo command line
    writes a folder of random weights from a config.json and samples from it."""
    import json
    import os
    import subprocess
    import sys
    from transformers_neuronx_b200 import NeuronAutoModelForCausalLM, TaboraxForSampling
    m = _model("A")
    model = NeuronAutoModelForCausalLM.from_pretrained(m.folder, batch_size=2, amp="f32", n_positions=64)
    assert isinstance(model, TaboraxForSampling)
    model.to_neuron()
    prompts = torch.tensor([m.random_ids(9, 41), m.random_ids(9, 42)])
    seq = model.sample(prompts, sequence_length=20, top_k=1)
    assert tuple(seq.shape) == (2, 20) and torch.equal(seq[:, :9], prompts)
    for row in seq.tolist():
        logits = m.plain_logits(row)
        for i in range(9, 20):
            lg = logits[i - 1]
            if row[i] != int(lg.argmax()):
                assert float(lg.max() - lg[row[i]]) / float(lg.abs().max()) <= 1e-4
                break
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    demo = os.path.join(root, "bin", "taborax_demo")
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(CONFIG_A))
    folder = tmp_path / "model"
    r = subprocess.run([sys.executable, demo, "--amp", "bf16", "save", str(folder), "--random", "--config", str(cfg)],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    r = subprocess.run([sys.executable, demo, "--amp", "bf16", "run", str(folder), "--batch_size", "2", "--n_positions", "24",
                        "--top_k", "1"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0 and "generated_sequence=" in r.stdout, r.stderr
