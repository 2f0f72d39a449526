"""Plain, slow restatement of the Lilenex design in torch on the CPU: one function per mechanism, whole sequences only
(no cache, no portions, which is the point: the framework's scheduled runs are compared with it).
Test infrastructure: nothing under cake_b200/ imports it and it imports nothing from there.

Notation: X [streams, S, W] residual streams, h [S, W] the input of a sublayer.  The model is a plain dict ``cfg`` (the parsed
config.json) and a dict ``wt`` name -> tensor.  ``dt`` is the torch dtype the arithmetic runs in (float32, or float64 for a
sharper bar)."""
import math

import torch

# tests only: a name from a test's list of planted mistakes, so that a test can show that its model would notice the mistake
FAULT = None


def lin(W, x):
    return x @ W.to(x.dtype).t()


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w.to(x.dtype)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


# ---- residual streams -------------------------------------------------------------------------------------------------
def read_streams(X, w):
    """u = sum_s w[s] X[s]"""
    return torch.einsum("s,stw->tw", w.to(X.dtype), X)


def write_streams(X, mix, out, y, mult):
    """X'[t] = sum_s mix[s, t] X[s] + mult out[t] y, every stream from the old ones"""
    if FAULT == "mix transposed":
        mix = mix.t()
    return torch.einsum("st,snw->tnw", mix.to(X.dtype), X) + (mult * out.to(X.dtype))[:, None, None] * y[None]


# ---- attention --------------------------------------------------------------------------------------------------------
def frequencies(rot):
    """(f_i for i < dims / 2, amplitude of cos and sin).  With ``scaling`` the pairs that turn less than ``slow`` times over ``original``
    positions are slowed by ``factor``, those that turn more than ``fast`` times keep their frequency, a linear ramp over the pair's
    index lies between."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, orig = float(sc["factor"]), float(sc["original"])

    def index_of(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(float(sc["fast"]))), 0)
    hi = min(math.ceil(index_of(float(sc["slow"]))), dims - 1)
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        f[i] = fi / factor * r + fi * (1.0 - r)
    return f, 0.1 * math.log(factor) + 1.0


def rotate(x, rot):
    """x [S, heads, dim], row = position: the first ``dims`` entries of every head turn in adjacent pairs, the rest pass."""
    if not rot or int(rot.get("dims") or 0) < 2:
        return x
    dims = int(rot["dims"])
    f, amp = frequencies(rot)
    if FAULT == "no amplitude":
        amp = 1.0
    ang = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)[None, :]
    c, s = (amp * torch.cos(ang)).to(x.dtype)[:, None, :], (amp * torch.sin(ang)).to(x.dtype)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y = x.clone()
    y[..., 0:dims:2], y[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return y


def window_mask(S, size, keep_first):
    """[S, S] bool: row i sees key j <= i when i - j < size or j < keep_first (size 0: every j <= i)."""
    i, j = torch.arange(S)[:, None], torch.arange(S)[None, :]
    if not size:
        return j <= i
    size += {"window+1": 1, "window-1": -1}.get(FAULT, 0)
    keep_first += {"keep+1": 1, "keep-1": -1}.get(FAULT, 0)
    if FAULT == "keep none":
        keep_first = 0
    return (j <= i) & ((i - j < size) | (j < keep_first))


def attend(q, k, v, vis, scale):
    """q [S, H, D], k [S, G, D], v [S, G, V], vis [S, S]: softmax attention, head h reads key head h / (H / G)."""
    r = q.shape[1] // k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(r, 1)) * scale
    p = torch.softmax(s.masked_fill(~vis[None], float("-inf")), -1)
    return torch.einsum("hij,jhv->ihv", p, v.repeat_interleave(r, 1))


def project_kv(h, wt, p, m, eps):
    """Keys (normed over the whole projection, then rotated) and values of a layer."""
    S, G = h.shape[0], int(m["kv_heads"])
    k = rms_norm(lin(wt[p + "k"], h), wt[p + "k.norm"], eps).view(S, G, int(m["dim"]))
    return rotate(k, m.get("rot")), lin(wt[p + "v"], h).view(S, G, int(m["vdim"]))


def attention(h, wt, p, m, eps, kv):
    S, H, D = h.shape[0], int(m["heads"]), int(m["dim"])
    q = lin(wt[p + "q"], h)
    if FAULT == "norm per head":
        q = rms_norm(q.view(S, H, D), wt[p + "q.norm"].view(H, D), eps)
    else:
        q = rms_norm(q, wt[p + "q.norm"], eps).view(S, H, D)
    mask = m.get("mask") or {}
    vis = window_mask(S, int(mask.get("size") or 0), int(mask.get("keep_first") or 0))
    o = attend(rotate(q, m.get("rot")), kv[0], kv[1], vis, float(m["scale"]))
    return lin(wt[p + "o"], o.reshape(S, -1))


# ---- gated linear attention --------------------------------------------------------------------------------------------
def gated_linear_attention(h, wt, p, m, eps):
    """S <- diag(a) S + k v^T, o = S^T q with a decay per key channel a = sigmoid(z)^(1 / tau) from a low-rank product; o of every head
    RMS-normed, heads times silu of a gate."""
    S, H, D, V = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (lin(wt[p + "q"], h) * D ** -0.5).view(S, H, D)
    k, v = lin(wt[p + "k"], h).view(S, H, D), lin(wt[p + "v"], h).view(S, H, V)
    z = lin(wt[p + "a2"], lin(wt[p + "a1"], h)) + wt[p + "a2.b"].to(h.dtype)
    a = torch.exp(torch.nn.functional.logsigmoid(z) / float(m["tau"])).view(S, H, D)
    if FAULT == "decay of the next channel":
        a = a.roll(1, -1)
    if FAULT == "no decay":
        a = torch.ones_like(a)
    st, out = torch.zeros(H, D, V, dtype=h.dtype), []
    for t in range(S):
        st = a[t][:, :, None] * st + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", st, q[t]))
    o = rms_norm(torch.stack(out), wt[p + "norm"], eps).reshape(S, H * V)
    return lin(wt[p + "o"], o * silu(lin(wt[p + "g"], h)))


# ---- feed-forwards -----------------------------------------------------------------------------------------------------
def dense_ff(h, wt, p):
    return lin(wt[p + "down"], gelu_tanh(lin(wt[p + "up"], h)))


def expert(h, wt, p):
    return lin(wt[p + "down"], silu(lin(wt[p + "gate"], h)) * lin(wt[p + "up"], h))


def route(z, top):
    """z [S, E] router logits -> (experts [S, top], weights [S, top]): the largest sigmoid scores (chosen by logit, which orders them
    where their rounded values are equal), as they are."""
    idx = torch.topk(z, top, -1).indices
    w = torch.sigmoid(torch.gather(z, 1, idx))
    if FAULT == "renormalised":
        w = w / w.sum(-1, keepdim=True)
    return idx, w


def routed_ff(h, wt, p, mlp):
    """The weight of a chosen expert scales its input."""
    r = mlp["router"]
    idx, w = route(lin(wt[p + "router"], h), int(r["top"]))
    y = torch.zeros_like(h)
    for e in range(int(r["experts"])):
        rows, slot = (idx == e).nonzero(as_tuple=True)
        if len(rows):
            g = w[rows, slot][:, None]
            y[rows] = y[rows] + (g * expert(h[rows], wt, f"{p}e{e}.") if FAULT == "weight behind" else expert(g * h[rows], wt, f"{p}e{e}."))
    if mlp.get("shared"):
        y = y + expert(h, wt, p + "shared.")
    return y


# ---- the model -----------------------------------------------------------------------------------------------------------
def layer(X, wt, cfg, i, kvs):
    L, p, eps, mult = cfg["layers"][i], f"l{i}.", float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    m = L["mixer"]

    def mixer(h):
        if L["type"] == "gla":
            return gated_linear_attention(h, wt, p + "mix.", m, eps)
        src = m.get("kv_from")
        if src is None:
            kvs[i] = project_kv(h, wt, p + "mix.", m, eps)
        return attention(h, wt, p + "mix.", m, eps, kvs[i if src is None else int(src)])

    def ff(h):
        return dense_ff(h, wt, p + "mlp.") if L["mlp"]["kind"] == "dense" else routed_ff(h, wt, p + "mlp.", L["mlp"])

    for q, f in ((1, mixer), (2, ff if L.get("mlp") is not None else None)):
        if f is not None:
            h = rms_norm(read_streams(X, wt[f"{p}hc{q}.in"]), wt[f"{p}norm{q}"], eps)
            X = write_streams(X, wt[f"{p}hc{q}.mix"], wt[f"{p}hc{q}.out"], f(h), mult)
    return X


def forward(tokens, wt, cfg, dt=torch.float32, trace=None):
    """Logits [S, vocab]; ``trace`` (a list) receives the sum of the streams after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = wt["embed"].to(dt)[torch.as_tensor(tokens, dtype=torch.long)]
    X, kvs = x[None].repeat(int(cfg["streams"]), 1, 1), {}
    for i in range(len(cfg["layers"])):
        X = layer(X, wt, cfg, i, kvs)
        if trace is not None:
            trace.append(X.sum(0))
    return lin(wt["embed"], rms_norm(X.sum(0), wt["final.norm"], eps))
