"""The Resatar decoder on the GPU against the plain implementation (tests/plain/resatar_plain.py): every mechanism's
kernel alone, then whole models through the replay program's function (whole prompts, token by token, portions down
to two tokens, mixed batches with pages and slots used again), keys just inside and outside a window and the tokens it keeps,
a distance bias that decides, decays that remember and forget, long decoding, and greedy generation through the engine's
own entry point and scheduler."""
import copy
import math
from types import SimpleNamespace

import pytest
import torch

from helpers import run_trace_inprocess
from plain import resatar_plain as RP
from vononex_helpers import BF16_WORST
from resatar_helpers import (CONFIG_A, CONFIGS, TOLERANCE, ResatarModel, attn, compare, cut_steps, dense, layer, left, mamba,
                             mixed_steps, moe, right, rot, side, whole_steps)

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64
_models = {}


def _model(name, seed=5):
    if (name, seed) not in _models:
        _models[(name, seed)] = ResatarModel(CONFIGS[name], seed=seed)
    return _models[(name, seed)]


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def _close(got, want, tol):
    err = float((got.double().cpu() - want.double()).abs().max()) / max(float(want.abs().max()), 1e-30)
    assert err <= tol, err


def _ctx(cuts, pad_rows=1):
    """cuts: per request (slot, first position, rows) -> the index arrays of a step, as the step function packs them,
    with a padded row and a padded request behind them."""
    req, pos, q_start, q_len, slots, row = [], [], [], [], [], 0
    for r, (slot, first, n) in enumerate(cuts):
        req += [r] * n
        pos += list(range(first, first + n))
        q_start.append(row); q_len.append(n); slots.append(slot)
        row += n
    return SimpleNamespace(token_request=_i32(req + [-1] * pad_rows), positions=_i32(pos + [0] * pad_rows),
                           q_start=_i32(q_start + [0]), q_len=_i32(q_len + [0]), state_slots=_i32(slots + [-1]),
                           decode_only=all(n == 1 for n in q_len))


# ---- attention kernels: a window that keeps the first tokens, a distance bias -----------------------
def _paged(k, v, window, keep, L, dtype, seed):
    """A cache that holds the keys and values [L, G, D] of one request on shuffled pages, with the pages between the kept
    tokens and the window of position L - 1 given back (-1 in the table)."""
    G, D = k.shape[1:]
    blocks = -(-L // 16)
    pages = torch.randperm(blocks + 3, generator=torch.Generator().manual_seed(seed))[:blocks].tolist()
    cache = torch.randn(blocks + 3, 2, G, 16, D, generator=torch.Generator().manual_seed(seed + 1)).to(dtype) * 3
    table = []
    for b in range(blocks):
        n = min(16, L - 16 * b)
        cache[pages[b], 0, :, :n] = k[16 * b:16 * b + n].transpose(0, 1).to(dtype)
        cache[pages[b], 1, :, :n] = v[16 * b:16 * b + n].transpose(0, 1).to(dtype)
        table.append(pages[b])
    return cache, table


def _drop_between(table, window, keep, first_query):
    """Blocks that no query from first_query on reads are given back."""
    if not window:
        return table
    return [p if 16 * b < keep or 16 * b + 15 > first_query - window else -1 for b, p in enumerate(table)]


def _sharp(H, G, D, L, dtype, seed, scale):
    """Queries and keys whose scores spread over about +-6, so that single keys decide a row."""
    g = torch.Generator().manual_seed(seed)
    q, k, v = torch.randn(L, H, D, generator=g), torch.randn(L, G, D, generator=g), torch.randn(L, G, D, generator=g)
    f = (6.0 / (scale * D ** 0.5)) ** 0.5          # scores of about +-6
    return (q * f).to(dtype), (k * f).to(dtype), v.to(dtype)


MASKS = [(0, 0), (37, 0), (37, 5), (16, 16), (64, 64), (1, 1), (100, 33), (48, 130), (130, 20), (2000, 7)]


def _plain_rows(q, k, v, scale, window, keep, r1, r2, rows):
    T = k.shape[0]
    bias = (lambda h: RP.distance_bias(T, float(r1[h]), float(r2[h]))) if r1 is not None else None
    o = RP.attend(q.double(), k.double(), v.double(), scale, RP.mask(T, window or None, keep), bias)
    return o[rows].reshape(len(rows), -1)


@pytest.mark.parametrize("with_bias", [False, True])
@pytest.mark.parametrize("window, keep", MASKS)
@pytest.mark.parametrize("H, G, D, dtype", [(4, 2, 32, torch.float32), (6, 3, 48, torch.bfloat16), (4, 1, 96, torch.bfloat16),
                                            (8, 2, 128, torch.bfloat16), (2, 2, 64, torch.bfloat16), (2, 1, 160, torch.bfloat16)])
def test_kept_tokens_and_the_distance_bias_in_prompts_and_decoding(H, G, D, dtype, window, keep, with_bias):
    """A context of 333 positions on shuffled pages (what lies between the kept tokens and the window is gone from the
    table): its last 201 rows as one portion, and single rows near the window's, a page's and the kept tokens' edges as
    decode rows with their own key appended by the kernel, under several splits of the context."""
    from transformers_neuronx_b200.kernels import ops
    L, scale = 333, 0.17
    q, k, v = _sharp(H, G, D, L, dtype, 11, scale)
    g = torch.Generator().manual_seed(12)
    r1 = r2 = bias = None
    if with_bias:
        r1, r2 = torch.rand(H, generator=g) * 2.0, torch.rand(H, generator=g) * 1.5
        r1[0], r2[-1] = 3.0, 20.0
        bias = (r1.to(DEV), r2.to(DEV))
    cache, table = _paged(k, v, window, keep, L, dtype, 13)
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    first = L - 201
    rows = list(range(first, L))
    want = _plain_rows(q, k, v, scale, window, keep, r1, r2, rows)
    dev = cache.to(DEV)
    bt = _i32([_drop_between(table, window, keep, first)])
    qs = q[first:].reshape(len(rows), H * D).contiguous().to(DEV)
    kw = dict(window=window, keep_first=keep, bias=bias)
    out = torch.empty_like(qs)
    if dtype == torch.float32:
        ops.attention_simt(qs, dev, bt, _i32([0] * len(rows)), _i32(rows), out, H, scale, **kw)
        _close(out, want, tol)
    else:
        tiles = [0, 128]
        args = (qs, dev, bt, _i32([0] * len(tiles)), _i32(tiles), _i32([0]), _i32([len(rows)]), _i32([first]), out, H, scale)
        (ops.attention_prefill_tc if ops.attention_prefill_tc_supported(qs, dev, out) else ops.attention_prefill)(*args, **kw)
        _close(out, want, tol)
        out.zero_()
        ops.attention_prefill(*args, **kw)
        _close(out, want, tol)
        out.zero_()
        ops.attention_simt(qs, dev, bt, _i32([0] * len(rows)), _i32(rows), out, H, scale, **kw)
        _close(out, want, tol)
    if dtype == torch.float32:
        return
    # decode rows at their own lengths: requests that hold p + 1 positions, the last of which comes with the step
    ps = sorted({0, 4, 15, 16, 17, keep, max(window - 1, 0), window, window + 1, window + keep, 63, 64, 200, L - 1} & set(range(L)))
    want = _plain_rows(q, k, v, scale, window, keep, r1, r2, ps)
    tabs = [_drop_between(table, window, keep, p)[:p // 16 + 1] for p in ps]
    bt = _i32([t + [-1] * (-(-L // 16) - len(t)) for t in tabs])
    qs = q[ps].reshape(len(ps), H * D).contiguous().to(DEV)
    kn, vn = k[ps].reshape(len(ps), G * D).contiguous().to(DEV), v[ps].reshape(len(ps), G * D).contiguous().to(DEV)
    for plan in (dict(), dict(n_splits=1, warps=4), dict(n_splits=3, warps=4), dict(n_splits=7, warps=8), dict(grouped=True), dict(grouped=False)):
        out = torch.empty(len(ps), H * D, device=DEV, dtype=dtype)
        ops.attention_decode(qs, dev, bt, _i32(list(range(len(ps)))), _i32(ps), out, H, scale, max_kv_len=L, new_kv=(kn, vn), **kw, **plan)
        _close(out, want, tol)
        out.zero_()
        ops.attention_decode(qs, dev, bt, _i32(list(range(len(ps)))), _i32(ps), out, H, scale, max_kv_len=L, **kw, **plan)
        _close(out, want, tol)


def test_a_long_window_walks_more_pages_than_a_block_keeps_in_shared_memory():
    """2,300 keys behind kept tokens: more pages than the tensor-core prefill kernel lists in shared memory."""
    from transformers_neuronx_b200.kernels import ops
    H, G, D, L, scale, window, keep = 2, 1, 64, 3000, 0.2, 2300, 70
    q, k, v = _sharp(H, G, D, L, torch.bfloat16, 21, scale)
    cache, table = _paged(k, v, window, keep, L, torch.bfloat16, 22)
    first = L - 130
    rows = list(range(first, L))
    r1, r2 = torch.tensor([0.3, 1.2]), torch.tensor([0.5, 0.01])
    want = _plain_rows(q, k, v, scale, window, keep, r1, r2, rows)
    qs = q[first:].reshape(len(rows), H * D).contiguous().to(DEV)
    out = torch.empty_like(qs)
    ops.attention_prefill_tc(qs, cache.to(DEV), _i32([_drop_between(table, window, keep, first)]), _i32([0, 0]), _i32([0, 128]), _i32([0]),
                             _i32([len(rows)]), _i32([first]), out, H, scale, window=window, keep_first=keep,
                             bias=(r1.to(DEV), r2.to(DEV)))
    _close(out, want, 1.5e-2)


# ---- what lies around the attention kernels -----------------------------------------------------------
@pytest.mark.parametrize("H, G, dk, dv, rotary, norm, dtype", [
    (6, 2, 20, 28, (12, 1e4, (8.0, 1.5, 6.0, 64)), False, torch.float32), (4, 2, 96, 64, (96, 1e4, None), False, torch.bfloat16),
    (8, 2, 64, 64, (32, 1e5, (4.0, 1.0, 4.0, 128)), False, torch.bfloat16), (6, 3, 12, 20, None, True, torch.float32),
    (8, 2, 128, 128, None, True, torch.bfloat16), (1, 1, 50, 30, None, True, torch.float32)])
def test_queries_keys_and_mixed_values(H, G, dk, dv, rotary, norm, dtype):
    """Stretched rotation on part of a head, a norm over the whole projection, values mixed with another layer's (and not),
    the padding of a head, a padded row left alone."""
    from transformers_neuronx_b200.kernels import ops
    from transformers_neuronx_b200.parts.rotary import inverse_frequencies
    from transformers_neuronx_b200.parts.spec import FrequencyBandsSpec
    g = torch.Generator().manual_seed(3)
    D = -(-max(dk, dv) // 16) * 16
    pos = [0, 1, 63, 64, 700, 4095]
    T, nq, nk, nv = len(pos), H * dk, G * dk, G * dv
    width = nq + nk + nv
    proj = torch.zeros(T + 1, -(-width // 8) * 8, dtype=dtype)
    proj[:T, :width] = (torch.randn(T, width, generator=g) * 2).to(dtype)
    other = torch.randn(T + 1, nv + 8, generator=g).to(dtype)
    wq, wk = (torch.randn(nq, generator=g), torch.randn(nk, generator=g)) if norm else (None, None)
    u = proj[:T].double()
    q, k, v = u[:, :nq], u[:, nq:nq + nk], u[:, nq + nk:width]
    if norm:
        q, k = RP.rms(q, 1e-5, wq.double()), RP.rms(k, 1e-5, wk.double())
    q, k = q.reshape(T, H, dk), k.reshape(T, G, dk)
    inv = None
    if rotary:
        sc = dict(zip(("factor", "low", "high", "original"), rotary[2])) if rotary[2] else None
        q, k = RP.rotate(q, pos, rotary[0], rotary[1], sc), RP.rotate(k, pos, rotary[0], rotary[1], sc)
        inv = inverse_frequencies(rotary[0], rotary[1], DEV, FrequencyBandsSpec(**sc) if sc else None)
    tol = 3e-6 if dtype == torch.float32 else 5e-3
    dv_ = lambda t: None if t is None else t.to(DEV)
    for lam in (None, 0.3, -0.8):
        outs = [torch.full((T + 1, n), 9.0, device=DEV, dtype=dtype) for n in (H * D, G * D, G * D)]
        od = other.to(DEV)
        ops.rotary_qkv_prep(proj.to(DEV), 0, nq, nq + nk, _i32([0] * T + [-1]), _i32(pos + [0]), dv_(wq), dv_(wk), 1e-5, None, inv,
                            rotary[0] if rotary else 0, None, *outs, H, G, dk, dv, D,
                            other_values=od[:, 8:] if lam is not None else None,
                            mix_weight=torch.tensor([lam], device=DEV) if lam is not None else None)
        want_v = v if lam is None else (1 - lam) * v + lam * other[:T, 8:].double()
        qo, ko, vo = (o.float().cpu() for o in outs)
        for o in (qo, ko, vo):
            assert float((o[T] - 9.0).abs().max()) == 0.0
        for o, want, n, w in ((qo, q, H, dk), (ko, k, G, dk), (vo, want_v.reshape(T, G, dv), G, dv)):
            o = o[:T].reshape(T, n, D)
            _close(o[..., :w], want, tol)
            assert D == w or float(o[..., w:].abs().max()) == 0.0


@pytest.mark.parametrize("H, dv, D, dtype", [(6, 28, 32, torch.float32), (4, 64, 96, torch.bfloat16), (8, 128, 128, torch.bfloat16),
                                             (1, 30, 64, torch.bfloat16), (5, 20, 32, torch.float32)])
def test_gates_behind_the_attention(H, dv, D, dtype):
    from transformers_neuronx_b200.kernels import ops
    g = torch.Generator().manual_seed(4)
    T = 7
    att = torch.randn(T + 1, H * D, generator=g).to(dtype)
    a = att[:T].double().reshape(T, H, D)[..., :dv]
    tol = 3e-6 if dtype == torch.float32 else 5e-3
    for n in (H, H * dv):
        gate = (torch.randn(T + 1, -(-(n + 8) // 8) * 8, generator=g) * 2).to(dtype)
        f = torch.sigmoid(gate[:T, 8:8 + n].double())
        want = (a * (f[..., None] if n == H else f.reshape(T, H, dv)) * 1.3).reshape(T, H * dv)
        out = torch.full((T + 1, H * dv + 8), 9.0, device=DEV, dtype=dtype)
        gd = gate.to(DEV)
        ops.rotary_unrotate(att.to(DEV), _i32([0] * T + [-1]), _i32([5] * (T + 1)), None, 1.3, out[:, 8:], H, dv, D, gate=gd[:, 8:8 + n])
        _close(out[:T, 8:], want, tol)
        assert float((out[T].float() - 9.0).abs().max()) == 0.0 and float((out[:, :8].float() - 9.0).abs().max()) == 0.0


# ---- the two recurrences ------------------------------------------------------------------------------
CUTS = [(5, 1), (1, 2), (2, 0), (1, 1), (8, 17), (1, 1), (0, 1), (23, 18)]       # rows of two requests, step by step


def _walk(seqs, slots, cuts_list, step):
    """Runs `step(rows of the step [n + a padded one, width], ctx)` over the sequences cut as cuts_list says; returns the rows."""
    got, at = [[] for _ in seqs], [0] * len(seqs)
    for ns in cuts_list:
        reqs = [r for r, n in enumerate(ns) if n]
        cuts = [(slots[r], at[r], ns[r]) for r in reqs]
        x = torch.cat([seqs[r][at[r]:at[r] + ns[r]] for r in reqs] + [torch.zeros_like(seqs[0][:1])])
        y = step(x, _ctx(cuts)).float().cpu()
        row = 0
        for r, (_, _, n) in zip(reqs, cuts):
            got[r].append(y[row:row + n])
            row += n; at[r] += n
    return [torch.cat(g) for g in got]


@pytest.mark.parametrize("C, R, N, taps, states, dtype", [
    (60, 5, 18, 5, 0, torch.float32), (128, 8, 16, 4, 2, torch.float32), (128, 8, 16, 4, 4, torch.float32), (50, 1, 70, 1, 0, torch.float32),
    (30, 7, 3, 8, 0, torch.float32), (200, 8, 32, 3, 2, torch.float32), (136, 8, 8, 4, 2, torch.float32), (40, 4, 128, 2, 0, torch.float32),
    (24, 4, 200, 3, 0, torch.float32), (72, 8, 6, 4, 4, torch.float32), (256, 16, 16, 4, 0, torch.bfloat16)])
def test_the_selective_scan_across_cuts_and_slots(C, R, N, taps, states, dtype):
    """Two requests cut into unequal steps side by side (single tokens, pairs, a padded row, a request left out of a step):
    convolution with bias and silu, step sizes, decays per channel and state, skip and gate, against the plain recurrence over the whole
    sequences; a slot nobody uses stays as it is, and a request that takes a freed (zeroed) slot does not see what was there."""
    from transformers_neuronx_b200.kernels import ops
    g = torch.Generator().manual_seed(5)
    T, keep = 41, taps - 1
    rnd = lambda *s: torch.randn(*s, generator=g)
    w, b, D, a_log = rnd(C, taps) * 0.5, rnd(C) * 0.3, rnd(C), rnd(C, N)
    a_log[0], a_log[1] = -9.0, 3.0                                     # a channel that forgets almost nothing, one that forgets at once
    state = torch.zeros(4, C, N, device=DEV)
    conv = torch.zeros(4, keep, C, device=DEV, dtype=dtype) if keep else None
    state[1].fill_(7.0)
    a2 = (-torch.exp(a_log.double()) / math.log(2.0)).float().to(DEV)
    wd, bd, Dd = w.t().contiguous().to(DEV), b.to(DEV), D.to(DEV)

    def step(rows, ctx):
        n = rows.shape[0]
        rows = rows.to(DEV)
        proj, low, dt = rows[:, :2 * C].to(dtype), rows[:, 2 * C:2 * C + R + 2 * N].to(dtype).contiguous(), rows[:, -C:].contiguous()
        x = torch.full((n, C), 9.0, device=DEV, dtype=dtype)
        ops.causal_conv(proj, 0, wd, bd, taps, conv, ctx, "silu", x)
        y = torch.full((n, C), 9.0, device=DEV, dtype=dtype)
        ops.selective_scan(x, dt, low, R, R + N, a2, Dd, proj[:, C:], state, ctx, "silu", y)
        assert float((x[-1].float() - 9.0).abs().max()) == 0.0 and float((y[-1].float() - 9.0).abs().max()) == 0.0
        return torch.cat([x.float(), y.float()], 1)

    def plain(s):
        s = s.double()
        x = RP.silu(RP.causal_conv(s[:, :C], w.double(), b.double()))
        if dtype == torch.bfloat16:
            x = x.bfloat16().double()
        y, S = RP.scan(x, torch.nn.functional.softplus(s[:, -C:], threshold=1e9), -torch.exp(a_log.double()), s[:, 2 * C + R:2 * C + R + N], s[:, 2 * C + R + N:2 * C + R + 2 * N], D.double())
        return torch.cat([x, y * RP.silu(s[:, C:2 * C])], 1), S

    seqs = []
    for _ in range(3):
        s = torch.cat([rnd(T, 2 * C + R + 2 * N).to(dtype).float(), rnd(T, C) * 3 - 1.0], 1)          # step sizes before their softplus
        seqs.append(s)
    ops.selective_scan_force(states, dtype)
    try:
        tol = 2e-5 if dtype == torch.float32 else 1e-2
        got = _walk(seqs[:2], [2, 0], CUTS, step)
        for r in range(2):
            want, S = plain(seqs[r])
            _close(got[r][:, C:], want[:, C:], tol)
            _close(state[[2, 0][r]], S, tol)
            if dtype == torch.float32:
                _close(got[r][:, :C], want[:, :C], 2e-6)
        assert float((state[1] - 7.0).abs().max()) == 0.0
        if keep:
            _close(conv[2].float(), seqs[0][T - keep:, :C].double(), 0.0)   # the last projected values, oldest first
            conv[2].zero_()
        state[2].zero_()
        got = _walk([seqs[2]], [2], [(3,), (1,), (1,), (30,), (2,), (1,), (1,), (1,), (1,)], step)
        _close(got[0][:, C:], plain(seqs[2])[0][:, C:], tol)
    finally:
        ops.selective_scan_force(0, dtype)


@pytest.mark.parametrize("H, dk, dv, dtype", [(5, 18, 10, torch.float32), (1, 4, 30, torch.float32), (3, 7, 9, torch.float32),
                                              (4, 128, 64, torch.float32), (2, 64, 96, torch.bfloat16), (8, 32, 16, torch.bfloat16)])
def test_lightning_attention_across_cuts_and_slots(H, dk, dv, dtype):
    """Activations on queries, keys and values, a fixed decay per head, a norm over all heads together with its weight and a
    sigmoid gate, through the kernels of portions and of single tokens."""
    from transformers_neuronx_b200.parts.retention import Retention
    from transformers_neuronx_b200.parts.spec import LinearSpec, RetentionSpec
    g = torch.Generator().manual_seed(6)
    T, W = 41, 24
    decay = [0.3, 0.9, 0.99, 0.9999, 0.7, 0.5, 0.95, 0.999][:H]
    lin = lambda n, i, o: LinearSpec(i, o, n)
    spec = RetentionSpec(kind="retention", hidden=W, n_heads=H, k_dim=dk, v_dim=dv, decay=tuple(decay), q=lin("q", W, H * dk),
                         k=lin("k", W, H * dk), v=lin("v", W, H * dv), gate=lin("g", W, H * dv), out=lin("o", H * dv, W),
                         norm_eps=1e-5, activation="silu", gate_activation="sigmoid", joint_norm=True, out_norm="norm")
    part = Retention(spec)
    t = {n: (torch.randn(s, generator=g) * 0.4).to(dtype) for n, s in
         (("q", (H * dk, W)), ("k", (H * dk, W)), ("v", (H * dv, W)), ("g", (H * dv, W)), ("o", (W, H * dv)), ("norm", (H * dv,)))}
    part.load(t, torch.device(DEV), dtype)
    from transformers_neuronx_b200.parts.base import StepContext
    state = torch.zeros(4, H, dv, dk, device=DEV)
    state[1].fill_(7.0)

    def step(rows, sc):
        ctx = StepContext(torch.device(DEV), dtype)
        for k_, v_ in vars(sc).items():
            setattr(ctx, k_, v_)
        ctx.cache_id, ctx.storage = 0, SimpleNamespace(tensor=lambda _: state)
        out = torch.empty(rows.shape[0], W, device=DEV)
        part.forward(ctx, rows.to(DEV), out, accumulate=False)
        return out
    seqs = [torch.randn(T, W, generator=g).to(dtype) for _ in range(2)]
    got = _walk(seqs, [3, 0], CUTS, step)
    m = {"heads": H, "dim": dk, "vdim": dv, "decay": decay}
    for r in range(2):
        want = RP.lightning(seqs[r].double(), {k_: v_.double() for k_, v_ in t.items()}, "", m, 1e-5)
        _close(got[r], want, 2e-5 if dtype == torch.float32 else 3e-2)
    assert float((state[1] - 7.0).abs().max()) == 0.0


# ---- the feed-forwards ---------------------------------------------------------------------------------
@pytest.mark.parametrize("E, top, W, always", [(6, 3, 72, 0), (8, 2, 256, 1), (1, 1, 24, 1), (5, 5, 33, 0), (64, 8, 128, 2)])
def test_routing_by_biased_logits(E, top, W, always):
    """Choice and weights of the softmax over the chosen logits, with a bias that changes the choice, and the experts that
    every token takes behind the chosen ones."""
    from transformers_neuronx_b200.kernels import ops
    g = torch.Generator().manual_seed(7)
    N = 40
    h, router, b = torch.randn(N, W, generator=g), torch.randn(E, W, generator=g) * 0.4, torch.randn(E, generator=g) * 3
    want = RP.route(h.double(), {"router": router.double(), "router.b": b.double()}, "", top)
    if 1 < top < E:
        assert any(w[0] != v[0] for w, v in zip(want, RP.route(h.double(), {"router": router.double(), "router.b": 0 * b.double()}, "", top)))
    ids = torch.empty(N + 1, top + always, dtype=torch.int32, device=DEV)
    wts = torch.empty(N + 1, top + always, device=DEV)
    ops.moe_route(torch.cat([h, torch.zeros(1, W)]).to(DEV), router.to(DEV), _i32([0] * N + [-1]), ids, wts, top, softmax_scores=True,
                  renormalize=True, bias=b.to(DEV), always=always)
    assert ids[N].tolist() == [-1] * (top + always)
    for n, (e_want, w_want) in enumerate(want):
        assert ids[n].tolist() == e_want + [E + i for i in range(always)], n
        _close(wts[n, :top], w_want, 3e-6)
        assert wts[n, top:].tolist() == [1.0] * always


@pytest.mark.parametrize("E, top, ff, shared, W, N, dtype", [
    (6, 3, 20, 20, 72, 5, torch.float32), (6, 3, 20, 28, 72, 5, torch.float32), (8, 2, 128, 128, 256, 3, torch.bfloat16),
    (8, 2, 128, 128, 256, 300, torch.bfloat16), (4, 2, 96, 160, 256, 40, torch.bfloat16), (5, 2, 36, None, 100, 9, torch.bfloat16)])
def test_experts_with_a_shared_one(E, top, ff, shared, W, N, dtype):
    """A shared expert as wide as the others (one more expert of the grouped products) and of another width (a gated
    feed-forward behind them), added to what the chosen experts give."""
    from transformers_neuronx_b200.models.resatar import _feed_forward
    from transformers_neuronx_b200.parts import build_part
    from transformers_neuronx_b200.parts.base import StepContext
    g = torch.Generator().manual_seed(8)
    mlp = moe(E, top, ff, shared)
    part = build_part("feed_forward", _feed_forward("m", W, mlp))
    assert part.folded == (shared == ff)
    t = {s.name: (torch.randn(s.shape, generator=g) * 0.15).to(dtype) for s in part.tensor_specs()}
    part.load(t, torch.device(DEV), dtype)
    h = torch.randn(N, W, generator=g).to(dtype)
    want = RP.experts(h.double(), {k[2:]: v.double() for k, v in t.items()}, "", mlp)
    ctx = StepContext(torch.device(DEV), dtype)
    ctx.token_request = _i32([0] * N)
    for accumulate in (False, True):
        out = torch.full((N, W), 1.0, device=DEV)
        part.forward(ctx, h.to(DEV), out, accumulate=accumulate)
        _close(out, want + (1.0 if accumulate else 0.0), 1e-5 if dtype == torch.float32 else 2e-2)
        ctx.begin_entry()


@pytest.mark.parametrize("N, K, F", [(300, 128, 512), (130, 72, 88), (5, 256, 512), (1, 256, 512), (2048, 64, 1000)])
def test_gelu_behind_the_up_product(N, K, F):
    """The tanh form of gelu in the products' epilogues (whole tiles, ragged edges, few tokens), over inputs from far below to
    far above zero; results are 16-bit."""
    from transformers_neuronx_b200.parts.linear import Linear
    from transformers_neuronx_b200.parts.spec import LinearSpec
    g = torch.Generator().manual_seed(9)
    for dtype in (torch.bfloat16, torch.float32):
        lin = Linear(LinearSpec(K, F, "w"))
        w = (torch.randn(F, K, generator=g) * torch.logspace(-2, 0, F)[:, None]).to(dtype)
        lin.load({"w": w}, torch.device(DEV), dtype)
        a = torch.randn(N, K, generator=g).to(dtype)
        out = torch.empty(N, F, device=DEV, dtype=dtype)
        lin.forward(a.to(DEV), out, activation="gelu_new")
        want = RP.gelu_tanh(a.double() @ w.double().T)
        err = (out.cpu().double() - want).abs()
        tol = 2e-6 if dtype == torch.float32 else 2.0 ** -8
        assert float((err - tol * want.abs()).max()) <= (2e-5 if dtype == torch.float32 else 1e-4)


# ---- whole models through the replay program's function -------------------------------------------
LENGTHS = {"A": [1, 2, 17, 45, 130], "B": [3, 140, 300], "C": [3, 70, 41]}
# The rows' median error in bfloat16: A and C are narrow (72, 100), A routes 3 of 6 experts (a rounding now and then picks another
# expert for a token), and a norm behind every sublayer lifts a small result, rounding included, to the size of the
# stream's steps.  The 32-bit engine holds every row to 3e-5.
BF16_MEDIAN = {"A": 7e-2, "B": TOLERANCE["bfloat16"], "C": 4e-2}


def _tol(name, dtype):
    return BF16_MEDIAN[name] if dtype == "bfloat16" else None


def _requests(m, lengths, seed=100):
    return {f"r{i}": m.random_ids(n, seed=seed + i) for i, n in enumerate(lengths)}


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_the_stream_after_every_layer(name):
    """The residual stream after each layer against the plain one: the first wrong layer names the mechanism."""
    from transformers_neuronx_b200.engine.loading import load_model
    from transformers_neuronx_b200.engine.step import StepEntry, StepRunner
    m = _model(name)
    ids = m.random_ids(90, 11)
    want = m.plain_hidden(ids)                                          # [layers, T, width]
    model, _ = load_model(m.folder, "float32", verbose=False)
    runner = StepRunner(model, page_size=16, num_pages=8, max_slots=2, max_model_len=128, use_cuda_graphs=False)
    runner.add_request("a")
    with model.tap_hidden_states() as taps:
        runner.step([StepEntry("a", ids, [len(ids) - 1])])
        torch.cuda.synchronize()
        for run in range(want.shape[0]):
            _close(taps[f"entry{run}"][:len(ids)], want[run], 2e-5)
    runner.finish("a")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_whole_prompts(name, dtype):
    m = _model(name)
    reqs = _requests(m, LENGTHS[name])
    steps = whole_steps(reqs)
    compare(m, reqs, steps, run_trace_inprocess(m.folder, dtype, steps, 64 * 5), dtype, tol=_tol(name, dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_a_prefix_then_token_by_token(name, dtype):
    """Decoding through the pages and the states: the last 85 tokens one by one (each window passes over decoded tokens,
    pages between it and the kept tokens are given back meanwhile), the steps replayed from a captured graph."""
    m = _model(name)
    reqs = _requests(m, [n for n in LENGTHS[name] if n > 86])
    steps = cut_steps(reqs, [1000], tail=85)
    compare(m, reqs, steps, run_trace_inprocess(m.folder, dtype, steps, 64 * 5), dtype, tol=_tol(name, dtype))


@pytest.mark.parametrize("name", ["A", "C"])
def test_from_the_first_token_on_one_by_one(name):
    """The first positions: zeros before the start of the convolution, states that start at zero, a softmax over one key."""
    m = _model(name)
    reqs = _requests(m, [60])
    steps = cut_steps(reqs, [1])
    compare(m, reqs, steps, run_trace_inprocess(m.folder, "float32", steps, 64), "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_portions_of_changing_size_down_to_two_tokens(name, dtype):
    """Portions shorter than the convolution (2 and 3 tokens under 5 taps), portions that end one before, at and one
    behind a page's border, and a long one."""
    m = _model(name)
    reqs = _requests(m, LENGTHS[name][-2:])
    steps = cut_steps(reqs, [2, 33, 3, 16, 2, 17, 64, 5, 15, 130], tail=3)
    compare(m, reqs, steps, run_trace_inprocess(m.folder, dtype, steps, 64 * 5), dtype, tol=_tol(name, dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_mixed_batches_with_pages_and_slots_used_again(name, dtype):
    """More requests than the replay program has slots: a finished request's slot (recurrent states and the convolution's
    last inputs) and its pages go to the next request, and the pool holds no more than the live requests need."""
    m = _model(name)
    lengths = {"A": [90, 7, 33, 150, 12, 64, 5, 49, 2, 120, 31], "B": [150, 20, 70, 9, 200, 40, 33, 129, 18],
               "C": [70, 41, 3, 20, 90, 2, 33]}[name]
    reqs = _requests(m, lengths, seed=300)
    steps = mixed_steps(reqs, [9, 2, 31, 16, 5, 64, 3])
    most = sorted(-(-n // 64) * 64 for n in lengths)[-4:]
    compare(m, reqs, steps, run_trace_inprocess(m.folder, dtype, steps, sum(most)), dtype, tol=_tol(name, dtype))


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


# ---- single keys that decide, decays that remember and forget --------------------------------------
def _one(kind, mixer, mlp=None, width=64, vocab=97):
    return {"architecture": "Resatar", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "init_std": 0.3,
            "layers": [layer(kind, mixer, mlp)]}


def _edge_steps(reqs):
    return (whole_steps(reqs), cut_steps(reqs, [48, 47, 2, 49, 16, 15, 1, 64], tail=57),
            mixed_steps(reqs, [31, 2, 48, 17], decode_tail=51))


@pytest.mark.parametrize("window, keep", [(40, 6), (64, 16), (33, 0), (17, 50)])
def test_a_sharp_softmax_finds_the_same_key_at_a_windows_edges(window, keep):
    """A scale that makes the softmax over normalised queries and keys nearly one-hot, so that every row reads single values:
    hundreds of tokens back among the kept ones, just inside the window, across pages, in prompts and decoded.  A window
    that is one off or a kept token more or less picks another value: the plain logits move wholesale then."""
    mixer = side(left(4, 2, 16, 24, 2.5, (window, keep)), right(2, 8, 8, (0.9, 0.5)), 1.0, 0.1)
    edit = lambda t: t.update({"l0.mix.left.r1": t["l0.mix.left.r1"] * 0.3})
    m = ResatarModel(_one("parallel", mixer), seed=22, edit=edit)
    reqs = {"a": m.random_ids(300, 1), "b": m.random_ids(77, 2)}
    for steps in _edge_steps(reqs):
        compare(m, reqs, steps, run_trace_inprocess(m.folder, "float32", steps, 64 * 7), "float32", tol=2e-4)
    plain = m.plain_logits(reqs["a"])
    for size, first in ((window + 1, keep), (window - 1, keep), (window, keep + 1)) + (((window, keep - 1),) if keep else ()):
        other = copy.deepcopy(m.cfg_dict)
        other["layers"][0]["mixer"]["left"]["mask"] = {"size": size, "keep_first": first}
        off = (RP.forward(other, m.plain_tensors, reqs["a"]).float() - plain).abs().amax(-1) / plain.abs().amax(-1)
        assert int((off > 0.02).sum()) >= 3, (size, first)


def test_a_far_key_among_hundreds_in_full_attention():
    """Rotated queries and keys with a large scale: rows that single keys from anywhere in the sequence decide, with values that
    the second layer mixes with the first one's."""
    cfg = _one("attention", attn(4, 2, 16, 24, 2.0, rot(8, 1e4, (4.0, 1.0, 4.0, 64)), True))
    cfg["layers"].append(layer("attention", attn(6, 2, 12, 24, 2.0, rot(12, 100.0), True), dense(40)))
    m = ResatarModel(cfg, seed=24, edit=lambda t: t.update({"l1.mix.vmix": torch.tensor(0.6, dtype=torch.bfloat16)}))
    reqs = {"a": m.random_ids(260, 1), "b": m.random_ids(61, 2)}
    for steps in _edge_steps(reqs):
        compare(m, reqs, steps, run_trace_inprocess(m.folder, "float32", steps, 64 * 6), "float32", tol=2e-4)


def test_a_distance_bias_that_decides():
    """Rates from 0.01 to 50 and multipliers up to 6 on weak scores: heads that see almost only the last keys beside heads that see
    them all evenly, without a window and with one."""
    def edit(t):
        t["l0.mix.left.r1"] = torch.tensor([6.0, 0.5, 2.0, 0.0], dtype=torch.bfloat16)
        t["l0.mix.left.r2"] = torch.tensor([0.01, 50.0, 1.0, 3.0], dtype=torch.bfloat16)
    for mask in (None, (90, 3)):
        m = ResatarModel(_one("parallel", side(left(4, 1, 16, 16, 0.1, mask), right(1, 8, 8, (0.5,)), 1.0, 0.2)), seed=25, edit=edit)
        reqs = {"a": m.random_ids(280, 1), "b": m.random_ids(70, 2)}
        for steps in _edge_steps(reqs):
            compare(m, reqs, steps, run_trace_inprocess(m.folder, "float32", steps, 64 * 7), "float32", tol=5e-5)
            compare(m, reqs, steps, run_trace_inprocess(m.folder, "bfloat16", steps, 64 * 7), "bfloat16")


def test_slow_decays_remember_the_first_tokens_and_fast_ones_forget():
    """A rate of e^-12 keeps what the first tokens wrote for the whole prompt, a rate of e^3 with a large step wipes it within a
    token; a head's decay of 0.99999 beside one of 0.01."""
    def rates(t):
        a, b = t["l0.mix.A_log"].clone(), t["l0.mix.dt.b"].clone()
        a[:20], a[20:40], b[20:40] = -12.0, 3.0, 2.0
        t["l0.mix.A_log"], t["l0.mix.dt.b"] = a, b
    cfg = _one("mamba1", mamba(72, 6, 16, 3))
    cfg["layers"].append(layer("parallel", side(left(2, 1, 8, 8, 0.3, (9, 2)), right(2, 16, 24, (0.99999, 0.01)), 0.2, 1.0), None))
    m = ResatarModel(cfg, seed=23, edit=rates)
    reqs = {"a": m.random_ids(260, 3)}
    for steps in (whole_steps(reqs), cut_steps(reqs, [2, 50, 1, 17], tail=30)):
        compare(m, reqs, steps, run_trace_inprocess(m.folder, "float32", steps, 64 * 5), "float32", tol=5e-5)


def test_long_decoding():
    m = _model("A")
    reqs = _requests(m, [260], seed=700)
    steps = cut_steps(reqs, [4], tail=250)
    compare(m, reqs, steps, run_trace_inprocess(m.folder, "float32", steps, 64 * 5), "float32")


# ---- the engine's own entry point ------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(dtype):
    from transformers_neuronx_b200.config import EngineConfig
    from transformers_neuronx_b200.engine import LLMEngine, load_model
    m = _model("B")
    model, typed = load_model(m.folder, dtype, verbose=False)
    eng = LLMEngine(model, EngineConfig(dtype=dtype, max_num_seqs=3, max_batch_tokens=48, max_portion=20, max_tokens=640,
                                        max_model_len=256))
    prompts = [m.random_ids(n, 900 + n) for n in (37, 5, 110, 18)]
    outs = eng.generate(prompts, 12, stop_on_eos=False)
    gaps = []
    for prompt, out in zip(prompts, outs):
        assert len(out) == 12
        logits = m.plain_logits(list(prompt) + list(out))
        for i, tok in enumerate(out):
            lg = logits[len(prompt) - 1 + i]
            gaps.append(float(lg.max() - lg[tok]) / float(lg.abs().max()))       # 0: the plain argmax
    # A tie that rounding may decide either way; in bfloat16 a token whose candidate experts are within a few thousandths may
    # take the other one, which changes its row wholesale: such rows are few (as in `compare`).
    gaps.sort()
    few = 0 if dtype == "float32" else len(gaps) // 16
    assert gaps[-few - 1] <= 2 * TOLERANCE[dtype] and gaps[-1] <= (2 * TOLERANCE[dtype] if few == 0 else BF16_WORST), gaps[-6:]
    eng.runner.cache.check()
    assert eng.runner.cache.slots.num_free == 3


def test_the_entry_point_class_and_the_command_line(tmp_path):
    """config.json picks the entry-point class; greedy `sample` equals the plain argmax, teacher-forced; the demo
    command line writes a folder of random weights from a config.json and samples from it."""
    import json
    import os
    import subprocess
    import sys
    from transformers_neuronx_b200 import NeuronAutoModelForCausalLM, ResatarForSampling
    m = _model("A")
    model = NeuronAutoModelForCausalLM.from_pretrained(m.folder, batch_size=2, amp="f32", n_positions=64)
    assert isinstance(model, ResatarForSampling)
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
    demo = os.path.join(root, "bin", "resatar_demo")
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(CONFIG_A))
    folder = tmp_path / "model"
    r = subprocess.run([sys.executable, demo, "--amp", "bf16", "save", str(folder), "--random", "--config", str(cfg)],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    r = subprocess.run([sys.executable, demo, "--amp", "bf16", "run", str(folder), "--batch_size", "2", "--n_positions", "24",
                        "--top_k", "1"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0 and "generated_sequence=" in r.stdout, r.stderr
