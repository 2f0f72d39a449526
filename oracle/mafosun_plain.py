"""Plain, slow restatement of the Mafosun design in torch on the CPU: one function per mechanism, whole sequences only
(no cache, no portions, which is the point: the framework's scheduled runs are compared with it).
Test infrastructure: nothing under cake_b200/ imports it and it imports nothing from there.

Notation: x [S, W] residual stream.  The model is a plain dict ``cfg`` (the parsed config.json) and a dict ``wt`` name -> tensor.
``dt`` is the torch dtype the arithmetic runs in (float32, or float64 for a sharper bar)."""
import math

import torch

# tests only: a name from a test's list of planted mistakes, so that a test can show that its model would notice the mistake
FAULT = None


def lin(W, x):
    return x @ W.to(x.dtype).t()


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w.to(x.dtype)


def frequencies(rot):
    """f_i of a rotation over ``dims`` entries; with ``scaling``, long wavelengths are stretched by ``factor``, short ones are kept
    and the ones between ``original / high`` and ``original / low`` are interpolated by turns over ``original`` positions."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc:
        factor, low, high, orig = (float(sc[k]) for k in ("factor", "low", "high", "original"))
        for i, fi in enumerate(f):
            wave = 2.0 * math.pi / fi
            if wave < orig / high:
                continue
            if wave > orig / low:
                f[i] = fi / factor
            else:
                s = (orig / wave - low) / (high - low)
                f[i] = (1.0 - s) * fi / factor + s * fi
    return f


def rotate(x, rot, interleaved):
    """x [S, heads, dim], row = position: the first ``dims`` entries of every head turn in pairs, (2i, 2i + 1) when interleaved,
    else (i, i + dims / 2); the rest pass."""
    if not rot or int(rot.get("dims") or 0) < 2:
        return x
    dims = int(rot["dims"])
    ang = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(frequencies(rot), dtype=torch.float64)[None, :]
    c, s = torch.cos(ang).to(x.dtype)[:, None, :], torch.sin(ang).to(x.dtype)[:, None, :]
    y = x.clone()
    if interleaved:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        y[..., 0:dims:2], y[..., 1:dims:2] = u * c - v * s, v * c + u * s
    else:
        u, v = x[..., : dims // 2], x[..., dims // 2: dims]
        y[..., : dims // 2], y[..., dims // 2: dims] = u * c - v * s, v * c + u * s
    return y


def window_mask(S, size):
    """[S, S] bool: row i sees key j when 0 <= i - j < size (size 0: every j <= i)."""
    i, j = torch.arange(S)[:, None], torch.arange(S)[None, :]
    if FAULT == "window+1" and size:
        size = size + 1
    if FAULT == "window-1" and size:
        size = size - 1
    return (j <= i) & ((i - j < size) if size else torch.ones(1, dtype=torch.bool))


def chunk_mask(S, size):
    """[S, S] bool: row i sees key j <= i of its own chunk of ``size`` positions counted from position 0 (size 0: every j <= i)."""
    i, j = torch.arange(S)[:, None], torch.arange(S)[None, :]
    if not size:
        return j <= i
    if FAULT == "chunk+1":
        size = size + 1
    if FAULT == "no chunk":
        return j <= i
    return (j <= i) & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))


def pool_blocks(k, v, pool):
    """Means over the complete blocks of ``pool`` rows: k [S, G, D] -> [S // pool, G, D], v likewise."""
    n = k.shape[0] // pool
    return (k[: n * pool].reshape(n, pool, *k.shape[1:]).mean(1), v[: n * pool].reshape(n, pool, *v.shape[1:]).mean(1))


def pool_mask(S, n, pool, size):
    """[S, n] bool: row i sees block b when its last position is at least ``size`` back."""
    i, b = torch.arange(S)[:, None], torch.arange(n)[None, :]
    if FAULT == "pool late":
        return b * pool + pool <= i - size
    if FAULT == "pool early":
        return b * pool + pool - 2 <= i - size
    if FAULT == "no pool":
        return torch.zeros(S, n, dtype=torch.bool)
    return b * pool + pool - 1 <= i - size


def attend(q, keys, values, vis, scale, softcap, sink):
    """q [S, H, D], keys [N, G, D], values [N, G, V], vis [S, N]: softmax attention per head; ``sink`` puts a one (a score of zero
    without a value) into the denominator."""
    H, G = q.shape[1], keys.shape[1]
    kk, vv = keys.repeat_interleave(H // G, 1), values.repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    s = s.masked_fill(~vis[None], float("-inf"))
    top = s.max(-1).values
    if sink:
        top = torch.clamp(top, min=0.0)
    e = torch.exp(s - top[..., None])
    den = e.sum(-1)
    if sink:
        den = den + torch.exp(-top)
    return torch.einsum("hij,jhv->ihv", e / den[..., None], vv)


def pooled_attention(h, wt, p, m, eps):
    """Grouped-query attention with normed, rotated queries and keys, a soft cap, a sliding window, pooled blocks of the positions
    before the window in the same softmax, and a sink of score zero."""
    S, H, G, D, V = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms_norm(lin(wt[p + "q"], h).view(S, H, D), wt[p + "q.norm"], eps)
    k = rms_norm(lin(wt[p + "k"], h).view(S, G, D), wt[p + "k.norm"], eps)
    v = lin(wt[p + "v"], h).view(S, G, V)
    q, k = rotate(q, m.get("rot"), True), rotate(k, m.get("rot"), True)
    mask = m.get("mask") or {}
    size, pool = int(mask.get("size") or 0), int(mask.get("pool") or 0)
    keys, values, vis = k, v, window_mask(S, size)
    if size and pool:
        pk, pv = pool_blocks(k, v, pool)
        keys, values = torch.cat([pk, k]), torch.cat([pv, v])
        vis = torch.cat([pool_mask(S, pk.shape[0], pool, size), vis], 1)
    o = attend(q, keys, values, vis, float(m["scale"]), float(m.get("softcap") or 0.0), FAULT != "no sink")
    return lin(wt[p + "o"], o.reshape(S, H * V))


def chunk_attention(h, wt, p, m, eps):
    """Grouped-query attention inside chunks of fixed places: normed queries, keys and (without gain) values, no positions."""
    S, H, G, D, V = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms_norm(lin(wt[p + "q"], h).view(S, H, D), wt[p + "q.norm"], eps)
    k = rms_norm(lin(wt[p + "k"], h).view(S, G, D), wt[p + "k.norm"], eps)
    v = rms_unit(lin(wt[p + "v"], h).view(S, G, V), eps)
    o = attend(q, k, v, chunk_mask(S, int((m.get("mask") or {}).get("size") or 0)), float(m["scale"]), 0.0, False)
    return lin(wt[p + "o"], o.reshape(S, H * V))


def retention(h, wt, p, m, eps):
    """A matrix state per head that decays by a fixed factor: S <- d S + k v^T, o = S^T q, unit-RMS per head, silu gate."""
    S, H, D, V = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate(lin(wt[p + "q"], h).view(S, H, D), m.get("rot"), False)
    k = rotate(lin(wt[p + "k"], h).view(S, H, D), m.get("rot"), False) * D ** -0.5
    v = lin(wt[p + "v"], h).view(S, H, V)
    d = torch.tensor([float(z) for z in m["decay"]], dtype=h.dtype)[:, None, None]
    st, out = torch.zeros(H, D, V, dtype=h.dtype), []
    for t in range(S):
        st = d * st + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", st, q[t]))
    o = rms_unit(torch.stack(out), eps).reshape(S, H * V)
    g = lin(wt[p + "g"], h)
    return lin(wt[p + "o"], o * g * torch.sigmoid(g))


def mixer(h, wt, p, L, eps):
    m = L["mixer"]
    if L["type"] == "attention":
        return pooled_attention(h, wt, p, m, eps)
    return float(m["left_scale"]) * chunk_attention(h, wt, p + "left.", m["left"], eps) + \
        float(m["right_scale"]) * retention(h, wt, p + "right.", m["right"], eps)


def gated_ff(h, wt, p, act):
    return lin(wt[p + "down"], act(lin(wt[p + "gate"], h)) * lin(wt[p + "up"], h))


def route(z, top, groups):
    """z [S, E] router logits -> (experts [S, top], weights [S, top]): softmax over all experts; only the experts of the ``keep``
    groups with the largest best score may be chosen; the weights are the scores as they are."""
    s = torch.softmax(z, -1)
    c = s.clone()
    if groups:
        n, keep = int(groups["count"]), int(groups["keep"])
        best = s.view(s.shape[0], n, -1).max(-1).values
        kept = torch.zeros_like(best, dtype=torch.bool).scatter(1, torch.topk(best, keep, -1).indices, True)
        if FAULT == "no groups":
            kept[:] = True
        c = c.view(s.shape[0], n, -1).masked_fill(~kept[..., None], -1.0).view_as(s)
    idx = torch.topk(c, top, -1).indices
    w = torch.gather(s, 1, idx)
    return idx, (w / w.sum(-1, keepdim=True) if FAULT == "renormalised" else w)


def routed_ff(h, wt, p, mlp):
    r = mlp["router"]
    idx, w = route(lin(wt[p + "router"], h), int(r["top"]), r.get("groups"))
    silu = lambda z: z * torch.sigmoid(z)
    y = torch.zeros_like(h)
    for e in range(int(r["experts"])):
        rows, slot = (idx == e).nonzero(as_tuple=True)
        if len(rows):
            y[rows] = y[rows] + w[rows, slot][:, None] * gated_ff(h[rows], wt, f"{p}e{e}.", silu)
    return y


def layer(x, wt, cfg, i):
    L, p, eps = cfg["layers"][i], f"l{i}.", float(cfg["norm"]["eps"])
    x = x + rms_norm(mixer(x, wt, p + "mix.", L, eps), wt[p + "norm1"], eps)
    mlp = L.get("mlp")
    if mlp is not None:
        y = gated_ff(x, wt, p + "mlp.", torch.relu) if mlp["kind"] == "dense" else routed_ff(x, wt, p + "mlp.", mlp)
        x = x + rms_norm(y, wt[p + "norm2"], eps)
    return x


def forward(tokens, wt, cfg, dt=torch.float32, trace=None):
    """Logits [S, vocab]; ``trace`` (a list) receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = rms_norm(wt["embed"].to(dt)[torch.as_tensor(tokens, dtype=torch.long)], wt["embed.norm"], eps)
    for i in range(len(cfg["layers"])):
        x = layer(x, wt, cfg, i)
        if trace is not None:
            trace.append(x.clone())
    return lin(wt["embed"], rms_norm(x, wt["final.norm"], eps))
