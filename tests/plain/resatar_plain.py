"""A plain, slow implementation of the Resatar decoder in 64-bit: the oracle of the tests.

One function per mechanism, loops over tokens where a loop says it most directly, whole sequences only (no cache,
no state, no batches): the engine's answers under any cut of a request must equal these.  It shares no code with
the package.

  embedding      x_t = E[token_t]
  layer          x <- x + n1b(mixer(n1(x))),  x <- x + n2b(ff(n2(x)));  n(y) = g y / sqrt(mean(y^2) + eps), g ONE number
  mixers         `softmax_attention` (rotated by stretched frequencies, values mixed with an earlier layer's, a gate a head),
                 `selective_scan` (a decay per channel and state), `side_by_side` (`biased_window_attention` beside
                 `lightning`, each with a factor)
  feed-forward   down(gelu(up h)), or routed experts down(silu(gate h) * up h) plus a shared one
  head           n_final(x), then the output matrix
"""
import math

import torch

F64 = torch.float64


def f32(z):
    return float(torch.tensor(z, dtype=torch.float32))


def rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def frequencies(dims, base, scaling=None):
    """f_i = base^(-2i / dims); with scaling, by the wave length 2 pi / f: short waves stay, long ones are slowed by the
    factor, those between `original / high` and `original / low` are blended."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            wave = 2.0 * math.pi / f
            if wave < scaling["original"] / scaling["high"]:
                pass
            elif wave > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            else:
                s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def rotate(x, positions, dims, base, scaling=None):
    """x [T, heads, d]: dim i turns with dim i + dims/2 on the first `dims` dims.  The design forms angles in 32-bit, so
    the frequency and the angle are rounded to 32-bit here too."""
    y = x.clone()
    half = dims // 2
    for t, p in enumerate(positions):
        for i, f in enumerate(frequencies(dims, base, scaling)):
            a = f32(float(p) * f32(f))
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, :, i], x[t, :, i + half]
            y[t, :, i], y[t, :, i + half] = u * c - v * s, v * c + u * s
    return y


def attend(q, k, v, scale, see, bias=None):
    """q [T, H, d], k [T, G, d], v [T, G, e], see [T, T] -> [T, H, e];  bias(h) [T, T] is taken off the scores."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if bias is not None:
            s = s - bias(h)
        out[:, h] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, g]
    return out


def mask(T, window=None, keep=0):
    """[query i, key j]: j <= i, and with a window i - j < window or j among the first `keep`."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    return see if window is None else see & ((i - j < window) | (j < keep))


def softmax_attention(h, t, p, m, first_values=None):
    """Returns (output, this layer's values as projected).  `first_values`: those of the first mixing layer."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ t[p + "q"].T).reshape(T, H, m["dim"])
    k = (h @ t[p + "k"].T).reshape(T, G, m["dim"])
    own = (h @ t[p + "v"].T).reshape(T, G, m["vdim"])
    rot = m.get("rot")
    if rot is not None:
        q = rotate(q, range(T), rot["dims"], rot["base"], rot.get("scaling"))
        k = rotate(k, range(T), rot["dims"], rot["base"], rot.get("scaling"))
    v = own
    if m.get("v_mix") and first_values is not None:
        lam = t[p + "vmix"]
        v = (1.0 - lam) * own + lam * first_values
    o = attend(q, k, v, m["scale"], mask(T))
    o = o * torch.sigmoid(h @ t[p + "g"].T)[:, :, None]
    return o.reshape(T, H * m["vdim"]) @ t[p + "o"].T, own


def distance_bias(T, r1, r2):
    d = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0).to(F64)
    return r1 * torch.log(1.0 + r2 * d)


def biased_window_attention(h, t, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms(h @ t[p + "q"].T + t[p + "q.b"], eps, t[p + "q.norm"]).reshape(T, H, m["dim"])
    k = rms(h @ t[p + "k"].T + t[p + "k.b"], eps, t[p + "k.norm"]).reshape(T, G, m["dim"])
    v = (h @ t[p + "v"].T + t[p + "v.b"]).reshape(T, G, m["vdim"])
    bias = lambda hd: distance_bias(T, float(t[p + "r1"][hd]), float(t[p + "r2"][hd]))
    mk = m.get("mask") or {}
    o = attend(q, k, v, m["scale"], mask(T, mk.get("size"), mk.get("keep_first", 0)), bias)
    o = o.reshape(T, H * m["vdim"]) * torch.sigmoid(h @ t[p + "g"].T)
    return o @ t[p + "o"].T + t[p + "o.b"]


def lightning(h, t, p, m, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ t[p + "q"].T).reshape(T, H, d)
    k = silu(h @ t[p + "k"].T).reshape(T, H, d)
    v = silu(h @ t[p + "v"].T).reshape(T, H, e)
    o = torch.zeros(T, H, e, dtype=F64)
    for hd in range(H):
        S = torch.zeros(d, e, dtype=F64)
        for i in range(T):
            S = m["decay"][hd] * S + torch.outer(k[i, hd], v[i, hd])
            o[i, hd] = S.T @ q[i, hd]
    o = rms(o.reshape(T, H * e), eps, t[p + "norm"]) * torch.sigmoid(h @ t[p + "g"].T)
    return o @ t[p + "o"].T


def side_by_side(h, t, p, m, eps):
    return (m["left_scale"] * biased_window_attention(h, t, p + "left.", m["left"], eps)
            + m["right_scale"] * lightning(h, t, p + "right.", m["right"], eps))


def causal_conv(u, w, b):
    """u [T, C], w [C, taps] (last column weighs the current token): zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
        y[t] += b
    return y


def scan(x, dt, A, B, C, D):
    """x, dt [T, c]; A [c, n]; B, C [T, n]; D [c] -> y [T, c] and the state left behind [c, n]."""
    S = torch.zeros_like(A)
    y = torch.zeros_like(x)
    for i in range(x.shape[0]):
        S = torch.exp(dt[i][:, None] * A) * S + (dt[i] * x[i])[:, None] * B[i][None, :]
        y[i] = S @ C[i] + D * x[i]
    return y, S


def selective_scan(h, t, p, m):
    inner, R, N = m["inner"], m["dt_rank"], m["state"]
    u = h @ t[p + "in"].T
    x, z = u[:, :inner], u[:, inner:]
    x = silu(causal_conv(x, t[p + "conv"], t[p + "conv.b"]))
    low = x @ t[p + "x"].T
    dt = torch.nn.functional.softplus(low[:, :R] @ t[p + "dt"].T + t[p + "dt.b"], threshold=1e9)
    y, _ = scan(x, dt, -torch.exp(t[p + "A_log"]), low[:, R:R + N], low[:, R + N:], t[p + "D"])
    return (y * silu(z)) @ t[p + "o"].T


def dense(h, t, p):
    return gelu_tanh(h @ t[p + "up"].T) @ t[p + "down"].T


def gated(h, t, p):
    return (silu(h @ t[p + "gate"].T) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def route(h, t, p, top):
    """[(experts, weights)] per token: the largest logits, weights the softmax over the chosen logits only."""
    z = h @ t[p + "router"].T + t[p + "router.b"]
    out = []
    for i in range(h.shape[0]):
        ids = sorted(range(z.shape[1]), key=lambda e: (-float(z[i, e]), e))[:top]
        out.append((ids, torch.softmax(torch.stack([z[i, e] for e in ids]), 0)))
    return out


def experts(h, t, p, mlp):
    y = torch.zeros_like(h)
    for i, (ids, w) in enumerate(route(h, t, p, mlp["router"]["top"])):
        for e, we in zip(ids, w):
            y[i] += we * gated(h[i:i + 1], t, p + f"e{e}.")[0]
    if mlp.get("shared") is not None:
        y = y + gated(h, t, p + "shared.")
    return y


def forward(config, tensors, tokens, keep_layers=False):
    """Logits [T, vocab] of one whole sequence (and the stream after every layer with keep_layers)."""
    t = {k: v.to(F64) for k, v in tensors.items() if v.is_floating_point()}
    eps = config["norm"]["eps"]
    norm = lambda x, name: rms(x, eps) * t[name]
    x = t["embed"][torch.tensor(tokens)]
    first_values, stream = None, []
    for i, layer in enumerate(config["layers"]):
        p, m, kind = f"l{i}.", layer["mixer"], layer["type"]
        h = norm(x, p + "norm1")
        if kind == "attention":
            mix, own = softmax_attention(h, t, p + "mix.", m, first_values)
            if m.get("v_mix") and first_values is None:
                first_values = own
        elif kind == "mamba1":
            mix = selective_scan(h, t, p + "mix.", m)
        else:
            mix = side_by_side(h, t, p + "mix.", m, eps)
        x = x + norm(mix, p + "norm1b")
        mlp = layer.get("mlp")
        if mlp is not None:
            h = norm(x, p + "norm2")
            ff = dense(h, t, p + "mlp.") if mlp["kind"] == "dense" else experts(h, t, p + "mlp.", mlp)
            x = x + norm(ff, p + "norm2b")
        stream.append(x.clone())
    logits = norm(x, "final.norm") @ t["head"].T
    return (logits, stream) if keep_layers else logits
