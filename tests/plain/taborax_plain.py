"""A plain, slow implementation of the Taborax decoder in 64-bit: the oracle of the tests.

One function per mechanism, loops over heads and tokens where a loop says it most directly, whole sequences only (no
cache, no state, no batches): the engine's answers under any cut of a request must equal these.  It shares no code with
the package.

  embedding      x_t = E[token_t]; x0 is kept
  layer          x <- x + n1b(mixer(n1(x)));  x <- x + n2b(ff(n2(x)))     n(y) = g y / sqrt(mean(y^2) + eps)
  order          layers[0 .. start), then layers[start .. stop) `times` times (the same weights, every pass with a past
                 of its own, and x <- W_in [x; x0] ahead of each pass), then layers[stop ..)
  mixers         `latent_attention` (no positions, queries and keys/values through low-rank latents),
                 `sink_attention` (rotated halves, the values are the unrotated keys, softmax with an empty sink)
  feed-forward   `dense`: down(relu(up h)^2), or `experts`: a softmax router with a correction of the choice, groups,
                 experts that return their input, and a shared expert behind a gate
  head           n_final(x), then the output matrix
"""
import math

import torch

F64 = torch.float64


def rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


def turn(x, dims, base):
    """x [T, heads, d]: dim i turns with dim i + dims/2 by position * base^(-2i/dims), i < dims/2.  The design forms
    angles in 32-bit: frequency and angle are rounded to 32-bit here too, sine and cosine of that angle are 64-bit."""
    y = x.clone()
    half = dims // 2
    f32 = lambda z: float(torch.tensor(z, dtype=torch.float32))
    freq = [f32(float(base) ** (-2.0 * i / dims)) for i in range(half)]
    for p in range(x.shape[0]):
        for i in range(half):
            a = f32(float(p) * freq[i])
            c, s = math.cos(a), math.sin(a)
            u, v = x[p, :, i], x[p, :, i + half]
            y[p, :, i], y[p, :, i + half] = u * c - v * s, v * c + u * s
    return y


def causal(T):
    return torch.arange(T)[None, :] <= torch.arange(T)[:, None]


def softmax_rows(scores):
    """scores [T, T] (query, key): softmax over the keys up to the query's own position."""
    return torch.softmax(scores.masked_fill(~causal(scores.shape[0]), -math.inf), -1)


def softmax_with_sink(scores, sink=0.0):
    """p_ij = exp(s_ij) / (exp(sink) + sum_j exp(s_ij)): one more key of score `sink` that has no value."""
    T = scores.shape[0]
    s = scores.masked_fill(~causal(T), -math.inf)
    return torch.softmax(torch.cat([torch.full((T, 1), sink, dtype=F64), s], 1), -1)[:, 1:]


def latent_attention(h, t, p, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    cq = rms(h @ t[p + "dq"].T, eps, t[p + "dq.norm"])
    q = (cq @ t[p + "uq"].T).reshape(T, H, d)
    c = rms(h @ t[p + "dkv"].T, eps, t[p + "dkv.norm"])
    k = (c @ t[p + "uk"].T).reshape(T, H, d)
    v = (c @ t[p + "uv"].T).reshape(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=F64)
    for hd in range(H):
        out[:, hd] = softmax_rows((q[:, hd] @ k[:, hd].T) * float(m["scale"])) @ v[:, hd]
    return out.reshape(T, H * dv) @ t[p + "o"].T


def sink_attention(h, t, p, m):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ t[p + "q"].T).reshape(T, H, d)
    k = (h @ t[p + "k"].T).reshape(T, G, d)
    v = k
    rot = m.get("rot")
    if rot and rot.get("dims"):
        q, k = turn(q, rot["dims"], rot["base"]), turn(k, rot["dims"], rot["base"])
    out = torch.zeros(T, H, d, dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = softmax_with_sink((q[:, hd] @ k[:, g].T) * float(m["scale"])) @ v[:, g]
    return out.reshape(T, H * d) @ t[p + "o"].T


def dense(h, t, p):
    return torch.clamp(h @ t[p + "up"].T, min=0.0) ** 2 @ t[p + "down"].T


def gated(h, t, p):
    return (silu(h @ t[p + "gate"].T) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def choose(s, correction, top, groups=None):
    """The chosen outputs of one token, from its scores s [E] (a list of numbers): the largest of s + correction, of the
    best groups only; of equal ones the lowest index."""
    E = len(s)
    c = [float(s[e]) + (float(correction[e]) if correction is not None else 0.0) for e in range(E)]
    open_ = set(range(E))
    if groups:
        n = E // groups["count"]
        best = sorted(range(groups["count"]), key=lambda g: (-max(c[g * n:(g + 1) * n]), g))[:groups["keep"]]
        open_ = {e for g in best for e in range(g * n, (g + 1) * n)}
    return sorted(open_, key=lambda e: (-c[e], e))[:top]


def experts(h, t, p, mlp):
    r = mlp["router"]
    s = torch.softmax(h @ t[p + "router"].T, -1)
    y = torch.zeros_like(h)
    for i in range(h.shape[0]):
        for e in choose(s[i], t.get(p + "correction"), r["top"], r.get("groups")):
            o = h[i] if e >= r["experts"] else gated(h[i:i + 1], t, p + f"e{e}.")[0]
            y[i] += s[i, e] * o
    if mlp.get("shared") is not None:
        y = y + torch.sigmoid(h @ t[p + "shared.sg"].T) * gated(h, t, p + "shared.")
    return y


def walk(cfg):
    """[(layer, whether it begins a pass of the loop)] in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, False) for i in range(a)] + [(i, i == a) for i in range(a, b)] * loop["times"]
            + [(i, False) for i in range(b, n)])


def forward_hidden(ids, tensors, cfg):
    """The residual stream after every layer run, [runs, T, width], and the logits [T, vocab]."""
    t = {k: v.to(F64) for k, v in tensors.items()}
    eps = float(cfg["norm"]["eps"])
    norm = lambda y, name: rms(y, eps, t[name])
    x0 = x = t["embed"][list(ids)]
    after = []
    for i, begins in walk(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if begins:
            x = torch.cat([x, x0], -1) @ t["loop.in"].T
        h = norm(x, p + "norm1")
        if layer["type"] == "latent_attention":
            y = latent_attention(h, t, p + "mix.", layer["mixer"], eps)
        else:
            y = sink_attention(h, t, p + "mix.", layer["mixer"])
        x = x + norm(y, p + "norm1b")
        mlp = layer.get("mlp")
        if mlp is not None:
            h = norm(x, p + "norm2")
            y = dense(h, t, p + "mlp.") if mlp["kind"] == "dense" else experts(h, t, p + "mlp.", mlp)
            x = x + norm(y, p + "norm2b")
        after.append(x.clone())
    return torch.stack(after), norm(x, "final.norm") @ t["head"].T


def forward_logits(ids, tensors, cfg):
    return forward_hidden(ids, tensors, cfg)[1]
