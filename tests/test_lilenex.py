"""Lilenex (several residual streams mixed around every sublayer; windowed attention that keeps the first tokens, with norms over the
whole q / k projections, blended rotation frequencies and keys shared between layers; linear attention with a decay per key channel;
feed-forwards without a gate, or routed by sigmoid scores that weigh the experts' inputs) through the framework's own entry points
(Context, TextModelBase, Sessions, Master) against the plain restatement in oracle/lilenex_plain.py, on small configurations made here
with random weights.

What a schedule must not change: the logits at a position are the same whether the prompt went in whole, token by token or in
portions, whatever ran before in the same cache slot, and whatever other request is interleaved.  fp32 (D = float) is the sharp
comparison: the GPU and the plain code differ by summation order only.  The error of a position is the root mean square over
the vocabulary of the difference (mean removed) over the spread of the expected logits.  Where random weights would hide a
fault (a key at a window's edge, a kept token, a decay read from the wrong channel, a transposed mixing matrix) the test first shows
that the plain model with that fault differs by many tolerances, then that the framework agrees with the right one.
"""
import copy
import ctypes
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from cake_b200.config import Config
from cake_b200.synth import make_lilenex_checkpoint
from oracle import lilenex_plain as P

TOL = {"f32": 2e-4, "bf16": 1e-1, "f16": 2e-2}   # bf16 at widths of a few dozen: every projection is rounded to 8 bits
YARN = {"factor": 6.0, "fast": 8.0, "slow": 1.0, "original": 100}   # at base 200 and 8 entries: a ramp that keeps, blends and slows pairs


def dense(ff=24):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=12, shared=10):
    d = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    return dict(d, shared={"ff": shared}) if shared else d


def attn(heads=4, kv_heads=2, dim=12, vdim=10, size=7, keep=2, scale=0.4, rot=8, base=200.0, scaling=YARN, kv_from=None, mlp="dense"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size, "keep_first": keep} if size else None,
         "rot": ({"dims": rot, "base": base, "scaling": dict(scaling)} if scaling else {"dims": rot, "base": base}) if rot else None}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": dense() if mlp == "dense" else mlp}


def gla(heads=3, dim=8, vdim=12, tau=4.0, mlp="moe"):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": moe() if mlp == "moe" else mlp}


def make_config(layers, width=44, vocab=53, eps=1e-5, streams=2, mult=0.6) -> Config:
    return Config.from_hf(json.loads(json.dumps({"architecture": "Lilenex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "streams": streams,
                                                 "residual_mult": mult, "layers": layers})))


def full_config(**kw) -> Config:
    """Every mechanism, unequal sizes, one layer without a feed-forward, two layers that read an earlier layer's keys with masks of their own."""
    return make_config([attn(), gla(), attn(heads=6, size=4, keep=1, scale=0.6, kv_from=0, mlp=moe(5, 1, 16, 0)),
                        attn(heads=3, kv_heads=3, dim=9, vdim=16, size=10, keep=0, rot=4, scaling=None, mlp=moe(8, 3, 9, 14)),
                        gla(heads=2, dim=20, vdim=7, tau=16.0, mlp=None), attn(heads=2, size=0, kv_from=0, mlp=dense(30)), gla(heads=1, dim=4, vdim=40, mlp=dense(9))], **kw)


def tokens(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def errors(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape, (got.shape, want.shape)
    assert np.isfinite(got).all()
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / max(float(want.std()), 1e-3)


def close(got, want, dtype, what="", bar=None):
    e = errors(got, want)
    if dtype == "f32":
        assert e.max() < TOL[dtype], f"{what}: worst {e.max():.3g} at position {int(e.argmax())}"
    else:   # a router's close call may flip under 16-bit rounding
        bar = bar or TOL[dtype]
        assert np.quantile(e, 0.9) < bar and np.median(e) < bar / 2 and e.max() < max(6 * bar, 1.0), \
            f"{what}: median {np.median(e):.3g}, 90 % within {np.quantile(e, 0.9):.3g}, worst {e.max():.3g} (bar {bar:.3g})"


def plain(cfg, sd, toks, streams=None, fault=None):
    P.FAULT = fault
    try:
        return P.forward(toks, {k: v.float() for k, v in sd.items()}, cfg.to_hf(), torch.float32, streams).numpy()
    finally:
        P.FAULT = None


def plain_with_rounded_products(cfg, sd, toks, to=torch.bfloat16):
    """The plain model with the input and the result of every matrix product rounded to 16 bits: how far that rounding alone
    moves the logits of a configuration (a router's close call, a sharp softmax), which is the bar a 16-bit run is held to."""
    exact = P.lin
    P.lin = lambda W, x: exact(W, x.to(to).float()).to(to).float()
    try:
        return plain(cfg, sd, toks)
    finally:
        P.lin = exact


def bar16(cfg, sd, toks, want, dtype="bf16"):
    to = torch.bfloat16 if dtype == "bf16" else torch.float16
    return max(TOL[dtype], 2 * float(np.quantile(errors(plain_with_rounded_products(cfg, sd, toks, to), want), 0.95)))


class Runner:
    """The framework side: a model on the GPU and its Sessions."""

    def __init__(self, cfg, sd, dtype, max_seq=None):
        from cake_b200.model import Context, Sessions, TextModelBase
        self.ctx = Context(cfg, sd, dtype, device=0, max_seq=max_seq or cfg.max_seq_len)
        self.model = TextModelBase.load(self.ctx)
        self.ses = Sessions(self.model, max_seq or cfg.max_seq_len)

    def run(self, rid, toks, cuts=None, end=True):
        """Feed ``toks`` as request ``rid`` in portions of the sizes ``cuts`` (the last one repeats; None = whole) -> logits of every position."""
        out, p, i = [], 0, 0
        while p < len(toks):
            n = len(toks) - p if not cuts else min(cuts[min(i, len(cuts) - 1)], len(toks) - p)
            lg = self.ses.step(rid, toks[p:p + n], want=list(range(n)))
            self.ctx.sync()
            out.append(lg.cpu().numpy())
            p, i = p + n, i + 1
        if end:
            self.ses.end(rid)
        return np.concatenate(out, 0)

    def rows(self, rows, cuts, cap):
        """The batch rows ``rows`` (equal lengths) in one call per portion -> [rows, positions, vocab]."""
        from cake_b200.model import Cache
        B = len(rows)
        self.ctx.cache = Cache(self.ctx, B, cap)
        got, p = [], 0
        for n in cuts:
            lg = self.model.forward(np.array([t[p:p + n] for t in rows], dtype=np.uint32), p, want=list(range(B * n)))
            self.ctx.sync()
            got.append(lg.cpu().numpy().reshape(B, n, -1))
            p += n
        return np.concatenate(got, 1)

    def close(self):
        self.ctx.close()


# ---------------------------------------------------------------------------------------------- no GPU needed
def test_config_round_trip():
    cfg = full_config()
    d = cfg.to_hf()
    assert d["architecture"] == "Lilenex" and len(d["layers"]) == 7 and d["layers"][4]["mlp"] is None and d["layers"][2]["mixer"]["kv_from"] == 0
    back = Config.from_hf(json.loads(json.dumps(d)))
    assert back.layers == cfg.layers and back.layer_list and back.block_kind == "lilenex" and back.tie_word_embeddings
    assert (back.streams, back.stream_width) == (2, 88) and back.head_tensor_names() == ("embed", "final.norm", None)
    assert [i for i, _ in back.run_plan()] == list(range(7))
    a, g, s = back.layers[0], back.layers[1], back.layers[5]
    assert a.type == "sink_attention" and (a.window, a.keep_first, a.qk_norm_wide, a.kv_back, a.streams, a.residual_mult) == (7, 2, True, 0, 2, 0.6)
    assert a.rot.interleaved and (a.rot.factor, a.rot.fast, a.rot.slow, a.rot.original) == (6.0, 8.0, 1.0, 100) and (a.dense_act, a.dense_plain) == (1, True)
    assert g.type == "gated_linear" and g.decay_tau == 4.0 and (g.moe.sigmoid_scores, g.moe.weigh_input, g.moe.plain_weights, g.moe.shared_ff) == (True, True, True, 10)
    assert (s.kv_back, s.window, s.keep_first) == (5, 0, 0) and back.layers[3].rot.factor == 0.0 and back.layers[2].moe.shared_ff == 0
    for path, value in ((("layers", 0, "type"), "retention"), (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "rot", "dims"), 14),
                        (("layers", 0, "mlp", "kind"), "other"), (("layers", 1, "mixer", "tau"), 0.0), (("layers", 1, "mlp", "router", "top"), 7),
                        (("layers", 2, "mixer", "kv_from"), 1), (("layers", 2, "mixer", "kv_from"), 2), (("layers", 5, "mixer", "kv_from"), 2),
                        (("layers", 5, "mixer", "kv_from"), 3)):
        bad = json.loads(json.dumps(d))
        node = bad
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(ValueError):
            Config.from_hf(bad)
    one = make_config([attn(size=0, rot=0)], streams=None, mult=None)
    assert (one.streams, one.layers[0].residual_mult, one.layers[0].window, one.layers[0].rot.dims) == (1, 1.0, 0, 0)


def test_checkpoint_names_and_shapes():
    from cake_b200.loader import lilenex_block_tensors
    cfg = full_config()
    sd = make_lilenex_checkpoint(cfg, "bf16", seed=1)
    assert "head" not in sd and sd["final.norm"].shape == (44,)
    b = [lilenex_block_tensors(sd, cfg, i) for i in range(7)]
    assert b[0]["q_norm"].shape == (48,) and b[0]["k_norm"].shape == (24,) and b[0]["v"].shape == (20, 44) and b[0]["o"].shape == (44, 40)
    assert b[0]["hc1_mix"].shape == (2, 2) and b[0]["hc2_in"].shape == (2,) and b[0]["ff_up"].shape == (24, 44) and "ff_gate" not in b[0]
    assert "k" not in b[2] and "v" not in b[2] and "k_norm" not in b[2] and b[2]["q_norm"].shape == (72,) and "s_gate" not in b[2]
    assert b[1]["a1"].shape == (8, 44) and b[1]["a2"].shape == (24, 8) and b[1]["norm"].shape == (12,) and cfg.layers[1].decay_rank == 8
    assert len(b[1]["e_gate"]) == 6 and b[1]["s_down"].shape == (44, 10) and "norm2" not in b[4] and "hc2_in" not in b[4]
    bad = dict(sd)
    bad["l0.mix.k.norm"] = sd["l0.mix.k.norm"][:5]
    with pytest.raises(ValueError):
        lilenex_block_tensors(bad, cfg, 0)
    del bad["l1.hc2.mix"]
    with pytest.raises(KeyError):
        lilenex_block_tensors(bad, cfg, 1)
    one = make_config([attn()], streams=None)       # a plain residual sum: no coefficients in the checkpoint
    s1 = {k: v for k, v in make_lilenex_checkpoint(one, "bf16", seed=2).items() if ".hc" not in k}
    t = lilenex_block_tensors(s1, one, 0)
    assert t["hc1_mix"].tolist() == [[1.0]] and t["hc2_out"].tolist() == [1.0]


def test_plain_masks_and_rotation():
    w = P.window_mask(9, 3, 2)
    assert w[8].tolist() == [True, True] + [False] * 4 + [True] * 3 and w[1].tolist() == [True, True] + [False] * 7 and w[3].tolist() == [True] * 4 + [False] * 5
    assert P.window_mask(4, 0, 1)[3].all()
    f, amp1 = P.frequencies({"dims": 8, "base": 200.0})
    g, amp = P.frequencies({"dims": 8, "base": 200.0, "scaling": YARN})
    # 100 positions: pair 0 turns 15.9 times (above fast), the others 4.2, 1.1 and 0.3 times
    assert amp1 == 1.0 and abs(amp - (0.1 * np.log(6.0) + 1.0)) < 1e-12 and g[0] == f[0] and f[1] > g[1] > f[1] / 6 and f[2] > g[2] > f[2] / 6 and abs(g[3] - f[3] / 6) < 1e-15
    x = torch.randn(5, 2, 10, dtype=torch.float64)
    y = P.rotate(x, {"dims": 8, "base": 200.0})
    assert torch.allclose(y[..., 8:], x[..., 8:]) and torch.allclose(y[0], x[0]) and torch.allclose((y * y).sum(-1), (x * x).sum(-1))
    assert torch.allclose(y[3, 0, 2], x[3, 0, 2] * np.cos(3 * f[1]) - x[3, 0, 3] * np.sin(3 * f[1]))
    z = P.rotate(x, {"dims": 8, "base": 200.0, "scaling": YARN})
    assert torch.allclose((z * z)[..., :8].sum(-1), amp * amp * (x * x)[..., :8].sum(-1))


def test_plain_streams_and_router():
    X = torch.randn(2, 3, 4)
    mix, out, y = torch.tensor([[0.5, 2.0], [-1.0, 0.25]]), torch.tensor([3.0, -1.0]), torch.randn(3, 4)
    N = P.write_streams(X, mix, out, y, 0.5)
    assert torch.allclose(N[0], 0.5 * X[0] - 1.0 * X[1] + 1.5 * y) and torch.allclose(N[1], 2.0 * X[0] + 0.25 * X[1] - 0.5 * y)
    assert torch.allclose(P.read_streams(X, torch.tensor([2.0, -1.0])), 2 * X[0] - X[1])
    idx, w = P.route(torch.tensor([[1.0, -2.0, 0.5]]), 2)
    assert idx[0].tolist() == [0, 2] and torch.allclose(w[0], torch.sigmoid(torch.tensor([1.0, 0.5])))
    z = torch.linspace(-4, 4, 9)
    assert torch.allclose(P.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))


def test_plain_gated_linear_attention_is_a_decayed_sum():
    cfg = make_config([gla(mlp=None)])
    sd = {k: v.double() for k, v in make_lilenex_checkpoint(cfg, "f32", seed=3).items()}
    h = torch.randn(6, 44, dtype=torch.float64)
    q, k, v = (P.lin(sd[f"l0.mix.{n}"], h).view(6, 3, -1) for n in "qkv")
    a = (torch.sigmoid(P.lin(sd["l0.mix.a2"], P.lin(sd["l0.mix.a1"], h)) + sd["l0.mix.a2.b"]) ** 0.25).view(6, 3, 8)
    o = sum(((q[5] * 8 ** -0.5 * a[j + 1:].prod(0) * k[j]).sum(-1, keepdim=True) * v[j]) for j in range(6))
    o = P.rms_norm(o, sd["l0.mix.norm"], 1e-5).reshape(-1)
    want = P.lin(sd["l0.mix.o"], o * P.silu(P.lin(sd["l0.mix.g"], h)[5]))
    assert torch.allclose(P.gated_linear_attention(h, sd, "l0.mix.", cfg.to_hf()["layers"][0]["mixer"], 1e-5)[5], want)


# ---------------------------------------------------------------------------------------------- GPU
MECHANISMS = {
    "attention_plain": ([attn(size=0, rot=0, mlp=None)], {}),
    "attention_window": ([attn(size=5, keep=0, rot=0, mlp=None)], {}),
    "attention_window_of_one": ([attn(size=1, keep=3, mlp=None)], {}),
    "attention_keeps_more_than_its_window": ([attn(size=2, keep=9, mlp=None)], {}),
    "attention_full_rotation": ([attn(dim=12, rot=12, scaling=None, mlp=None)], {}),
    "attention_blended_rotation": ([attn(dim=16, rot=16, base=5000.0, scaling={"factor": 3.0, "fast": 4.0, "slow": 0.5, "original": 30}, mlp=None)], {}),
    "attention_blend_of_one_step": ([attn(dim=16, rot=6, base=30.0, scaling={"factor": 9.0, "fast": 1.0, "slow": 1.0, "original": 20}, mlp=None)], {}),
    "attention_every_head_its_keys": ([attn(heads=3, kv_heads=3, mlp=None)], {}),
    "attention_one_key_head": ([attn(heads=5, kv_heads=1, dim=20, vdim=36, rot=6, mlp=None)], {}),
    "attention_one_head": ([attn(heads=1, kv_heads=1, mlp=None)], {}),
    "attention_wide_heads": ([attn(heads=2, kv_heads=1, dim=72, vdim=136, rot=40, mlp=None)], {}),
    "attention_head_of_300": ([attn(heads=1, kv_heads=1, dim=300, vdim=20, rot=300, mlp=None)], {}),
    "shared_keys": ([attn(mlp=None), attn(heads=8, kv_from=0, mlp=None)], {}),
    "shared_keys_other_masks": ([gla(mlp=None), attn(size=3, keep=1, mlp=None), gla(mlp=None), attn(size=12, keep=0, scale=0.8, kv_from=1, mlp=None),
                                 attn(size=0, kv_from=1, mlp=None)], {}),
    "linear": ([gla(mlp=None)], {}),
    "linear_one_head": ([gla(heads=1, dim=5, vdim=7, tau=1.0, mlp=None)], {}),
    "linear_keys_of_32": ([gla(heads=2, dim=32, vdim=136, mlp=None)], {}),
    "linear_keys_of_36_values_of_20": ([gla(heads=2, dim=36, vdim=20, tau=0.5, mlp=None)], {}),
    "linear_keys_of_96_values_of_72": ([gla(heads=3, dim=96, vdim=72, tau=30.0, mlp=None)], {}),
    "linear_keys_of_128": ([gla(heads=1, dim=128, vdim=128, mlp=None)], {}),
    "linear_keys_of_200": ([gla(heads=1, dim=200, vdim=36, mlp=None)], {}),
    "linear_state_in_shared_memory": ([gla(heads=2, dim=30, vdim=42, mlp=None)], {}),
    "linear_keys_beyond_the_registers": ([gla(heads=1, dim=300, vdim=60, mlp=None)], {}),
    "dense": ([attn(size=0, rot=0, mlp=dense(56))], {}),
    "experts": ([attn(mlp=moe(shared=0))], {}),
    "experts_and_a_shared_one": ([attn(mlp=moe())], {}),
    "experts_top_one": ([attn(mlp=moe(experts=7, top=1))], {}),
    "experts_all": ([attn(mlp=moe(experts=4, top=4))], {}),
    "experts_many": ([attn(mlp=moe(experts=80, top=7, ff=8))], {}),
    "experts_one": ([attn(mlp=moe(experts=1, top=1, ff=20))], {}),
    "one_stream": ([attn(), gla()], dict(streams=1, mult=1.0)),
    "three_streams": ([attn(), gla()], dict(streams=3, mult=1.3)),
    "four_streams_odd_width": ([attn(), gla()], dict(streams=4, mult=0.25, width=45)),
    "five_streams": ([attn(), gla()], dict(streams=5)),
    "seven_streams": ([attn(), gla()], dict(streams=7, width=48)),
    "sixteen_streams": ([attn(), gla()], dict(streams=16)),
    "a_wide_stream": ([gla(heads=2, mlp=dense(8))], dict(width=1100)),
    "a_large_eps": ([attn(), gla()], dict(eps=0.3)),
}


@pytest.mark.gpu
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_each_mechanism_alone(name):
    cfg = make_config(MECHANISMS[name][0], **MECHANISMS[name][1])
    sd = make_lilenex_checkpoint(cfg, "f32", seed=sum(map(ord, name)) % 1000)
    toks = tokens(41, cfg.vocab_size, seed=3)
    want = plain(cfg, sd, toks)
    r = Runner(cfg, sd, "f32")
    try:
        close(r.run("a", toks), want, "f32", "whole")
        close(r.run("b", toks, cuts=[1]), want, "f32", "token by token")
        close(r.run("c", toks, cuts=[2, 5, 3, 7, 2]), want, "f32", "portions")
    finally:
        r.close()


@pytest.mark.gpu
def test_one_stream_without_coefficients_is_the_plain_residual_sum():
    cfg = make_config([attn(), gla()], streams=None, mult=0.5)
    sd = make_lilenex_checkpoint(cfg, "f32", seed=4)
    for k in list(sd):
        if ".hc" in k:
            sd[k] = torch.ones_like(sd[k])
    toks = tokens(30, cfg.vocab_size, seed=3)
    want = plain(cfg, sd, toks)
    r = Runner(cfg, {k: v for k, v in sd.items() if ".hc" not in k}, "f32")
    try:
        close(r.run("a", toks), want, "f32", "whole")
        close(r.run("c", toks, cuts=[2, 5, 1]), want, "f32", "portions")
    finally:
        r.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["f32", "f16"])
def test_residual_after_every_layer(dtype):
    """Blocks one call at a time (every block reads its first input out of the streams itself) and in one call (the block before has
    read it out); the sum of the streams after every layer."""
    from cake_b200.capi import check, lib, ptr
    cfg = full_config(streams=3)
    sd = make_lilenex_checkpoint(cfg, dtype, seed=5)
    toks = tokens(29, cfg.vocab_size, seed=4)
    streams = []
    plain(cfg, sd, toks, streams)
    r = Runner(cfg, sd, dtype)
    try:
        ctx, model = r.ctx, r.model
        for lo, hi in ((0, 17), (17, 29)):     # two portions: the second reads cache rows and state of the first in every layer
            ids = np.ascontiguousarray([toks[lo:hi]], dtype=np.uint32)
            x = ctx.empty(1, hi - lo, cfg.stream_width, dtype=torch.float32)
            check(lib().cake_b200_embed(ctx.h, ids.ctypes.data_as(ctypes.POINTER(ctypes.c_uint32)), 1, hi - lo, ptr(x)))
            for j, blk in enumerate(model.blocks):
                x = blk.forward_batch(x, [(blk.layer_name(), lo, j)], ctx, blocks=[blk])
                ctx.sync()
                want = streams[j][lo:hi].numpy()
                d = np.abs(x[0].cpu().numpy().reshape(hi - lo, 3, -1).sum(1) - want).max(-1)
                bar = (2e-4 if dtype == "f32" else 3e-2) * max(1.0, np.abs(want).max())
                assert (d.max() if dtype == "f32" else np.quantile(d, 0.9)) < bar, f"layer {j}, tokens {lo}..{hi}: {d.max():.3g}"
        assert len(model.blocks) == len(streams) == 7
    finally:
        r.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["f32", "bf16", "f16"])
def test_schedules_agree_with_the_plain_model(dtype):
    cfg = full_config()
    sd = make_lilenex_checkpoint(cfg, dtype, seed=11)
    toks = tokens(83, cfg.vocab_size, seed=5)
    want = plain(cfg, sd, toks)
    bar = None if dtype == "f32" else bar16(cfg, sd, toks, want, dtype)
    r = Runner(cfg, sd, dtype)
    try:
        whole = r.run("w", toks)
        close(whole, want, dtype, "whole", bar)
        for cuts in ([1], [2], [2, 3, 5], [17], [16, 16, 15, 1], [64, 1], [1, 40, 2]):
            got = r.run("c", toks, cuts=cuts)
            close(got, want, dtype, f"portions {cuts}", bar)
            if dtype == "f32":
                assert errors(got, whole).max() < TOL["f32"], f"portions {cuts} against whole"
        close(r.run("one", toks[:1]), want[:1], dtype, "a sequence of one token", bar)
        close(r.run("few", toks[:3], cuts=[1]), want[:3], dtype, "the first tokens", bar)
    finally:
        r.close()


@pytest.mark.gpu
def test_interleaved_requests_and_reused_slots():
    cfg = full_config()
    sd = make_lilenex_checkpoint(cfg, "f32", seed=21)
    a, b, c = tokens(50, cfg.vocab_size, seed=6), tokens(31, cfg.vocab_size, seed=7), tokens(64, cfg.vocab_size, seed=8)
    wa, wb, wc = plain(cfg, sd, a), plain(cfg, sd, b), plain(cfg, sd, c)
    r = Runner(cfg, sd, "f32")
    try:
        ga, gb, pa, pb = [], [], 0, 0
        for na, nb in ((7, 3), (1, 1), (20, 9), (2, 18), (20, 0)):      # two unequal requests, step by step in turns
            if na:
                ga.append(r.ses.step("a", a[pa:pa + na], want=list(range(na))).cpu().numpy())
                pa += na
            if nb:
                gb.append(r.ses.step("b", b[pb:pb + nb], want=list(range(nb))).cpu().numpy())
                pb += nb
        r.ses.end("a")
        r.ses.end("b")
        close(np.concatenate(ga), wa, "f32", "request a beside b")
        close(np.concatenate(gb), wb, "f32", "request b beside a")
        assert len(r.ses.free) == 2
        close(r.run("c", c, cuts=[9, 1]), wc, "f32", "a longer request in a used slot")    # rows and states of the old request lie there
        close(r.run("d", b, cuts=[4]), wb, "f32", "a shorter request in a used slot")
        close(r.run("e", a), wa, "f32", "whole in a used slot")
        assert len(r.ses.free) == 2 and not r.ses.live
    finally:
        r.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_batch_rows_against_each_alone(dtype):
    cfg = full_config()
    sd = make_lilenex_checkpoint(cfg, dtype, seed=31)
    rows = [tokens(40, cfg.vocab_size, seed=20 + i) for i in range(3)]
    want = [plain(cfg, sd, t) for t in rows]
    r = Runner(cfg, sd, dtype)
    try:
        got = r.rows(rows, (23, 1, 1, 15), 64)
        for i in range(3):
            close(got[i], want[i], dtype, f"batch row {i}", None if dtype == "f32" else bar16(cfg, sd, rows[i], want[i]))
    finally:
        r.close()


def show_faults(cfg, sd, toks, want, names, bar):
    for f in names:
        e = errors(plain(cfg, sd, toks, fault=f), want)
        assert e.max() > bar, f"{f} would not show: {e.max():.3g}"


@pytest.mark.gpu
@pytest.mark.parametrize("shared", [False, True])
def test_edges_of_windows_and_kept_tokens(shared):
    """Sharp scores, so that single keys carry a row.  A window one position longer or shorter, one kept token more or less or none: each
    changes the plain model's logits by many tolerances; the framework agrees with the right one in a whole prompt, in portions cut at
    and around every edge, and token by token.  With shared keys the second layer's window is wider than that of the layer whose keys it reads."""
    second = attn(size=13, keep=4, scale=0.9, kv_from=0, mlp=None) if shared else attn(heads=2, kv_heads=1, size=6, keep=1, scale=1.2, rot=4, mlp=dense())
    cfg = make_config([attn(size=11, keep=3, scale=1.0, mlp=None), second])
    sd = make_lilenex_checkpoint(cfg, "f32", seed=41)
    toks = tokens(90, cfg.vocab_size, seed=9)
    want = plain(cfg, sd, toks)
    show_faults(cfg, sd, toks, want, ("window+1", "window-1", "keep+1", "keep-1", "keep none"), 50 * TOL["f32"])
    r = Runner(cfg, sd, "f32")
    try:
        close(r.run("w", toks), want, "f32", "whole")
        for cuts in ([11], [10], [12], [13], [14], [6, 5], [1], [2], [3] + [1] * 12 + [9], [40, 2]):
            close(r.run("c", toks, cuts=cuts), want, "f32", f"portions {cuts}")
    finally:
        r.close()
    sb = {k: v.to(torch.bfloat16) for k, v in sd.items()}
    wb = plain(cfg, sb, toks)
    bar = bar16(cfg, sb, toks, wb)
    rb = Runner(cfg, sb, "bf16")
    try:
        close(rb.run("w", toks), wb, "bf16", "whole, bf16", bar)
        close(rb.run("c", toks, cuts=[30, 1]), wb, "bf16", "decoded, bf16", bar)
    finally:
        rb.close()


@pytest.mark.gpu
def test_faults_of_the_other_mechanisms_would_show():
    cfg = full_config()
    sd = make_lilenex_checkpoint(cfg, "f32", seed=44)
    toks = tokens(60, cfg.vocab_size, seed=19)
    want = plain(cfg, sd, toks)
    show_faults(cfg, sd, toks, want, ("mix transposed", "norm per head", "no amplitude", "decay of the next channel", "no decay", "renormalised", "weight behind"), 50 * TOL["f32"])
    r = Runner(cfg, sd, "f32")
    try:
        close(r.run("w", toks), want, "f32", "whole")
        close(r.run("c", toks, cuts=[9, 1, 1, 4]), want, "f32", "portions")
    finally:
        r.close()


def f16_case(layers, width, vocab, n, seed, faults):
    """A configuration in f16 (where rounding is small) with flat scores, so that every edge fault moves most positions: -> (cfg, sd,
    toks, want, bar) after showing that each fault would be seen."""
    cfg = make_config(layers, width=width, vocab=vocab)
    sd = make_lilenex_checkpoint(cfg, "f16", seed=seed)
    toks = tokens(n, vocab, seed=13)
    want = plain(cfg, sd, toks)
    bar = max(4 * float(np.quantile(errors(plain_with_rounded_products(cfg, sd, toks, torch.float16), want), 0.95)), 3e-3)
    for f in faults:
        e = errors(plain(cfg, sd, toks, fault=f), want)
        assert np.quantile(e, 0.5) > 2 * bar or e.max() > 12 * bar, f"{f} would not show: {np.quantile(e, 0.5):.3g}, {e.max():.3g} against {bar:.3g}"
    return cfg, sd, toks, want, bar


@pytest.mark.gpu
def test_key_size_128_portions_on_the_tensor_core_attention():
    """Key and value size 128 in 16-bit D: portions of 64 rows and more take the tensor-core attention (kept first tokens ahead of the
    window's tiles; a layer that shares keys), shorter ones the other kernels."""
    layers = [attn(heads=2, kv_heads=1, dim=128, vdim=128, size=9, keep=2, scale=0.02, rot=64, base=1000.0, scaling=None, mlp=None),
              attn(heads=4, kv_heads=1, dim=128, vdim=128, size=70, keep=5, scale=0.02, rot=64, base=1000.0, scaling=None, kv_from=0, mlp=dense(128)),
              gla(heads=2, dim=64, vdim=128, mlp=dense(128)),
              attn(heads=4, kv_heads=2, dim=128, vdim=128, size=130, keep=0, scale=0.02, rot=128, mlp=None)]
    cfg, sd, toks, want, bar = f16_case(layers, 128, 96, 500, 47, ("window+1", "window-1", "keep+1", "keep-1", "keep none", "decay of the next channel"))
    r = Runner(cfg, sd, "f16")
    try:
        whole = r.run("w", toks)
        close(whole, want, "f16", "whole", bar)
        for cuts in ([200, 130, 70], [64, 65, 128, 143], [37], [150, 1, 1, 1, 100, 2, 145]):
            got = r.run("c", toks, cuts=cuts)
            close(got, want, "f16", f"portions {cuts}", bar)
            close(got, whole, "f16", f"portions {cuts} against whole", bar)
        rows = [toks[:300], tokens(300, cfg.vocab_size, seed=14)]     # two batch rows in one call, in two portions
        wants = [want[:300], plain(cfg, sd, rows[1])]
        got = r.rows(rows, (200, 100), 320)
        for i in range(2):
            close(got[i], wants[i], "f16", f"batch row {i}", bar)
    finally:
        r.close()


@pytest.mark.gpu
def test_tiled_attention_of_other_head_sizes():
    """16-bit portions whose head sizes are multiples of eight but not 128, unequal for keys and values: the tiled kernel."""
    layers = [attn(heads=2, kv_heads=1, dim=24, vdim=40, size=9, keep=2, scale=0.05, rot=16, base=1000.0, scaling=None, mlp=None),
              attn(heads=4, kv_heads=1, dim=24, vdim=40, size=80, keep=1, scale=0.05, rot=16, base=1000.0, scaling=None, kv_from=0, mlp=dense(64)),
              gla(heads=2, dim=40, vdim=72, mlp=moe(8, 2, 64, 64)), attn(heads=3, kv_heads=3, dim=96, vdim=96, size=65, keep=70, scale=0.05, rot=96, mlp=None)]
    cfg, sd, toks, want, bar = f16_case(layers, 128, 128, 330, 48, ("window+1", "window-1", "keep+1", "keep-1", "keep none"))
    r = Runner(cfg, sd, "f16")
    try:
        whole = r.run("w", toks)
        close(whole, want, "f16", "whole", bar)
        for cuts in ([200, 130], [64, 66], [37], [150, 1, 1, 1, 100, 2]):
            close(r.run("c", toks, cuts=cuts), want, "f16", f"portions {cuts}", bar)
    finally:
        r.close()


@pytest.mark.gpu
def test_a_far_token_carries_weight():
    """One token's queries look for another token's keys: a kept first token and a plain key 430 positions back (over more than 256
    visible keys the split-key kernels run) decide the row; and a state that hardly decays remembers a token from far back."""
    cfg = make_config([attn(heads=2, kv_heads=2, dim=16, vdim=16, size=40, keep=3, scale=1.0, rot=4, base=1e6, scaling=None, mlp=None),
                       attn(heads=2, kv_heads=2, dim=16, vdim=16, size=0, scale=1.0, rot=4, base=1e6, scaling=None, kv_from=0, mlp=None)])
    sd = make_lilenex_checkpoint(cfg, "f32", seed=43)
    ask, answer = 7, 9
    sd["l0.norm1"] = torch.ones_like(sd["l0.norm1"])
    e = sd["embed"] / sd["embed"].pow(2).mean(-1, keepdim=True).sqrt()
    if float(sd["l0.hc1.in"].sum()) < 0:
        sd["l0.hc1.in"] = -sd["l0.hc1.in"]
    u = (e[ask] - e[answer]) / (e[ask] - e[answer]).norm()
    sd["l0.mix.q"] = sd["l0.mix.k"] @ (torch.eye(44) - 2 * u[:, None] * u[None, :])     # swaps the two embeddings, then looks for keys
    sd["l0.mix.q.norm"] = sd["l0.mix.k.norm"].clone()
    toks = [t if t not in (ask, answer) else 8 for t in tokens(460, cfg.vocab_size, seed=10)]
    toks[2], toks[455] = answer, ask
    want = plain(cfg, sd, toks)
    other = list(toks)
    other[2] = 3
    assert errors(plain(cfg, sd, other), want)[455] > 50 * TOL["f32"]      # the far token decides the row
    show_faults(cfg, sd, toks, want, ("keep none", "keep-1"), 50 * TOL["f32"])
    r = Runner(cfg, sd, "f32")
    try:
        close(r.run("w", toks), want, "f32", "whole")
        close(r.run("c", toks, cuts=[129, 127, 2, 1, 60]), want, "f32", "portions")
        close(r.run("d", toks, cuts=[400] + [1] * 60), want, "f32", "decoded")
    finally:
        r.close()
    slow = make_config([gla(heads=2, dim=16, vdim=16, tau=500.0, mlp=None)])
    ss = make_lilenex_checkpoint(slow, "f32", seed=43)
    want = plain(slow, ss, toks)
    assert errors(plain(slow, ss, other), want)[400:].max() > 20 * TOL["f32"]      # the state still holds the token
    r = Runner(slow, ss, "f32")
    try:
        close(r.run("w", toks), want, "f32", "whole, state")
        close(r.run("d", toks, cuts=[129, 127, 2] + [1] * 210), want, "f32", "decoded, state")
    finally:
        r.close()


@pytest.mark.gpu
def test_long_decoding_past_every_window():
    cfg = full_config()
    sd = make_lilenex_checkpoint(cfg, "f32", seed=45)
    toks = tokens(230, cfg.vocab_size, seed=11)
    want = plain(cfg, sd, toks)
    r = Runner(cfg, sd, "f32")
    try:
        close(r.run("d", toks, cuts=[10] + [1] * 220), want, "f32", "a short prompt then long decoding")
    finally:
        r.close()


@pytest.mark.gpu
def test_a_cache_that_the_request_fills_to_the_last_row():
    from cake_b200.capi import CakeB200Error
    cfg = full_config()
    sd = make_lilenex_checkpoint(cfg, "f32", seed=46)
    toks = tokens(31, cfg.vocab_size, seed=15)
    want = plain(cfg, sd, toks)
    r = Runner(cfg, sd, "f32", max_seq=31)
    try:
        close(r.run("w", toks), want, "f32", "whole")
        close(r.run("c", toks, cuts=[7, 1]), want, "f32", "portions")
        r.run("full", toks, end=False)
        with pytest.raises(CakeB200Error):
            r.ses.step("full", [1], want=[0])
        r.ses.end("full")
    finally:
        r.close()


@pytest.mark.gpu
def test_strong_decays_and_saturated_routers():
    """Decays near zero and near one side by side, router logits far into the sigmoid's tails."""
    cfg = make_config([gla(heads=2, dim=32, vdim=32, tau=1.0, mlp=moe()), gla(heads=2, dim=12, vdim=10, tau=0.25, mlp=None)])
    sd = make_lilenex_checkpoint(cfg, "f32", seed=49)
    for i in (0, 1):
        n = sd[f"l{i}.mix.a2.b"].numel()
        sd[f"l{i}.mix.a2.b"] = torch.linspace(-30.0, 30.0, n)
    sd["l0.mlp.router"] = sd["l0.mlp.router"] * 12.0      # several scores round to one: the logits decide
    toks = tokens(50, cfg.vocab_size, seed=16)
    want = plain(cfg, sd, toks)
    h = torch.randn(400, 44)
    assert ((torch.sigmoid(P.lin(sd["l0.mlp.router"], h)) == 1.0).sum(-1) > 2).any()
    r = Runner(cfg, sd, "f32")
    try:
        close(r.run("w", toks), want, "f32", "whole")
        close(r.run("c", toks, cuts=[19, 2, 1]), want, "f32", "portions")
    finally:
        r.close()


@pytest.mark.gpu
def test_other_sizes_and_tensor_core_shapes():
    """Sizes whose projections and experts take the tensor-core kernels (multiples of 128 / 64) next to ones that do not; long
    portions and decoding; against the plain model and whole against portions."""
    layers = [attn(heads=4, kv_heads=2, dim=64, vdim=64, size=96, keep=8, scale=0.1, rot=32, base=1000.0, mlp=dense(128)),
              gla(heads=4, dim=32, vdim=64, mlp=moe(6, 2, 64, 128)),
              attn(heads=2, kv_heads=2, dim=64, vdim=64, size=40, keep=1, scale=0.1, rot=32, base=1000.0, kv_from=0, mlp=moe(8, 3, 128, 64)),
              gla(heads=2, dim=24, vdim=20, mlp=dense(72))]
    cfg = make_config(layers, width=128, vocab=256, streams=4)
    toks = tokens(300, cfg.vocab_size, seed=12)
    for dtype in ("bf16", "f32"):
        sd = make_lilenex_checkpoint(cfg, dtype, seed=51)
        want = plain(cfg, sd, toks)
        # 16 bits: twice what rounding the products alone does to this configuration (its routed layers flip experts)
        bar = 2 * float(np.quantile(errors(plain_with_rounded_products(cfg, sd, toks), want), 0.95)) if dtype == "bf16" else None
        r = Runner(cfg, sd, dtype)
        try:
            whole = r.run("w", toks)
            close(whole, want, dtype, "whole", bar)
            got = r.run("c", toks, cuts=[133, 2, 1, 150, 1])
            close(got, want, dtype, "portions", bar)
            close(got, whole, dtype, "portions against whole", bar)
            close(r.run("d", toks, cuts=[260] + [1] * 40), want, dtype, "decoded", bar)
        finally:
            r.close()
    # without routers no position has an excuse: all of them within twice the worst that rounding the products causes
    for L in layers:
        L["mlp"] = dense(64)
    cfg = make_config(layers, width=128, vocab=256, streams=4)
    sd = make_lilenex_checkpoint(cfg, "bf16", seed=53)
    want = plain(cfg, sd, toks)
    bar = 2 * errors(plain_with_rounded_products(cfg, sd, toks), want).max()
    r = Runner(cfg, sd, "bf16")
    try:
        for cuts in (None, [133, 2, 1, 150, 1], [260] + [1] * 40):
            e = errors(r.run("w", toks, cuts=cuts), want)
            assert e.max() < bar, f"portions {cuts}: {e.max():.3g} at {int(e.argmax())} (bar {bar:.3g})"
    finally:
        r.close()


@pytest.mark.gpu
def test_refused_combinations():
    """Parts that are not built together are refused with a message, not computed wrongly."""
    from cake_b200.capi import CakeB200Error
    cfg = make_config([gla(), attn(), attn(kv_from=1)])
    sd = make_lilenex_checkpoint(cfg, "f32", seed=52)
    for layer, edit in ((0, dict(streams=3)), (0, dict(decay_tau=0.0)), (1, dict(norm_kind=1)), (1, dict(pool=2)), (1, dict(qk_unit=True)),
                        (1, dict(v_unit=True)), (2, dict(pool=3, keep_first=0))):
        bad = copy.deepcopy(cfg)
        for k, v in edit.items():
            setattr(bad.layers[layer], k, v)
        with pytest.raises((CakeB200Error, ValueError)):
            Runner(bad, sd, "f32")
    r = Runner(cfg, sd, "f32")
    try:    # a layer whose shared keys have not seen this step's positions: an error, and the step can still be made
        ctx, blocks = r.ctx, r.model.blocks
        x = torch.zeros(1, 4, cfg.stream_width, device="cuda")
        torch.cuda.synchronize()
        with pytest.raises(CakeB200Error):
            blocks[2].forward_batch(x, [(blocks[2].layer_name(), 0, 2)], ctx, blocks=[blocks[2]])
        for j in range(2):
            blocks[j].forward_batch(x, [(blocks[j].layer_name(), 0, j)], ctx, blocks=[blocks[j]])
        blocks[2].forward_batch(x, [(blocks[2].layer_name(), 0, 2)], ctx, blocks=[blocks[2]])
        with pytest.raises(CakeB200Error):
            blocks[2].forward_batch(x, [(blocks[2].layer_name(), 4, 2)], ctx, blocks=[blocks[2]])
        ctx.sync()
    finally:
        r.close()


@pytest.mark.gpu
def test_greedy_generation_through_master():
    from cake_b200.model import Context, Master, TextModelBase
    cfg = full_config()
    sd = make_lilenex_checkpoint(cfg, "f32", seed=61)
    prompt = tokens(9, cfg.vocab_size, seed=12)
    ctx = Context(cfg, sd, "f32", device=0, max_seq=64)
    try:
        out = Master(TextModelBase.load(ctx)).generate_text(prompt, 12)["tokens"]
    finally:
        ctx.close()
    seq = list(prompt)
    for tok in out:   # every generated token is the plain model's greedy choice, or within a hair of it
        lg = plain(cfg, sd, seq)[-1]
        assert lg[tok] >= lg.max() - 1e-2 * np.abs(lg).max(), (len(seq), tok, int(lg.argmax()))   # the sampler reads 16-bit logits
        seq.append(tok)
    assert len(out) == 12


@pytest.mark.gpu
def test_checkpoint_on_disk_through_the_trace_replayer_and_the_generate_command(tmp_path):
    """config.json + model.safetensors on disk -> `bin/trace_run` (steps on standard input, logits as files) and
    `python -m cake_b200.run` (token ids out): the model class follows the config in both."""
    from cake_b200.loader import open_model, save_checkpoint
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = full_config()
    sd = make_lilenex_checkpoint(cfg, "bf16", seed=81)
    model_dir, out_dir = str(tmp_path / "model"), str(tmp_path / "out")
    save_checkpoint(model_dir, cfg, sd)
    back, vb = open_model(model_dir)
    assert set(vb.keys()) == set(sd.keys()) and back.block_kind == "lilenex"
    toks = tokens(21, cfg.vocab_size, seed=14)
    want = plain(cfg, sd, toks)
    steps = [{"step": 0, "entries": [{"id": "r", "tokens": toks[:9], "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "r", "tokens": toks[9:11], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "r", "tokens": toks[11:], "want": [9]}], "end": ["r"]},
             {"step": 3, "entries": [{"id": "s", "tokens": toks[:4], "want": [3]}], "end": ["s"]}]
    for dtype in ("float32", "bfloat16"):
        res = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", model_dir, "--dtype", dtype, "--out", out_dir, "--max-tokens", "40"],
                             input="".join(json.dumps(x) + "\n" for x in steps), capture_output=True, text=True, timeout=900)
        assert res.returncode == 0, res.stderr[-2000:]
        assert [ln for ln in res.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        assert not os.path.exists(os.path.join(out_dir, "1.f32"))
        got = {i: np.fromfile(os.path.join(out_dir, f"{i}.f32"), dtype="<f4").reshape(-1, cfg.vocab_size) for i in (0, 2, 3)}
        short = "f32" if dtype == "float32" else "bf16"
        close(np.concatenate([got[0], got[2], got[3]]), want[[0, 8, 20, 3]], short, f"trace replay in {dtype}", 0.2)
    res = subprocess.run([sys.executable, "-m", "cake_b200.run", model_dir, "--prompt-ids", ",".join(map(str, toks[:6])), "-n", "5", "--dtype", "f32"],
                         capture_output=True, text=True, timeout=900, cwd=root)
    assert res.returncode == 0, res.stderr[-2000:]
    out = [int(t) for t in res.stdout.split("tokens:")[1].splitlines()[0].split()]
    assert len(out) == 5 and all(0 <= t < cfg.vocab_size for t in out)
