"""Mafosun (sublayers that read the stream itself and are normed on their output; grouped-query attention with pooled blocks in front
of its window, a soft cap and a sink of score zero; chunked attention beside retention; relu and group-limited routed
feed-forwards) through the framework's own entry points (Context, TextModelBase, Sessions, Master) against the plain restatement in
oracle/mafosun_plain.py, on small configurations made here with random weights.

What a schedule must not change: the logits at a position are the same whether the prompt went in whole, token by token or in
portions, whatever ran before in the same cache slot, and whatever other request is interleaved.  fp32 (D = float) is the sharp
comparison: the GPU and the plain code differ by summation order only.  The error of a position is the root mean square over
the vocabulary of the difference (mean removed) over the spread of the expected logits.  Where random weights would hide a
fault (a key at a window's edge, a pooled block that is one position early, the sink, a chunk's edge) the test first shows that
the plain model with that fault differs by many tolerances, then that the framework agrees with the right one.
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
from cake_b200.synth import make_mafosun_checkpoint
from oracle import mafosun_plain as P

TOL = {"f32": 2e-4, "bf16": 1e-1, "f16": 2e-2}   # bf16 at widths of a few dozen: every projection is rounded to 8 bits
STRETCH = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 40}   # at base 200 and 8 entries: one pair kept, one between, two stretched


def dense(ff=24):
    return {"kind": "dense", "ff": ff}


def moe(experts=12, top=3, ff=12, groups=3, keep=2):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}, "expert": {"ff": ff}}


def attn(heads=4, kv_heads=2, dim=12, vdim=10, size=7, pool=3, scale=0.7, softcap=5.0, rot=8, base=200.0, scaling=STRETCH, mlp="dense"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
         "mask": {"size": size, "pool": pool} if size else None,
         "rot": ({"dims": rot, "base": base, "scaling": dict(scaling)} if scaling else {"dims": rot, "base": base}) if rot else None}
    return {"type": "attention", "mixer": m, "mlp": dense() if mlp == "dense" else mlp}


def par(heads=6, kv_heads=3, dim=8, vdim=14, size=11, scale=0.6, ls=0.7, rheads=3, rdim=10, rvdim=6, rot=6, base=50.0, rs=0.4, decay=None, mlp="moe"):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size} if size else None}
    right = {"heads": rheads, "dim": rdim, "vdim": rvdim, "decay": decay or [1.0 - 2.0 ** -(2 + i) for i in range(rheads)],
             "rot": {"dims": rot, "base": base} if rot else None}
    return {"type": "parallel", "mixer": {"left": left, "left_scale": ls, "right": right, "right_scale": rs}, "mlp": moe() if mlp == "moe" else mlp}


def make_config(layers, width=44, vocab=53, eps=1e-5) -> Config:
    return Config.from_hf(json.loads(json.dumps({"architecture": "Mafosun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers})))


def full_config(**kw) -> Config:
    """Every mechanism, unequal sizes, one layer without a feed-forward."""
    return make_config([par(), attn(), attn(heads=3, kv_heads=3, dim=9, vdim=16, size=10, pool=5, softcap=2.0, rot=4, scaling=None, mlp=moe(8, 2, 16, 4, 1)),
                        par(heads=2, kv_heads=1, dim=20, vdim=8, size=5, rheads=2, rdim=8, rvdim=12, rot=8, mlp=None), par(size=17, mlp=dense(30))], **kw)


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


class Runner:
    """The framework side: a model on the GPU and its Sessions."""

    def __init__(self, cfg, sd, dtype, max_seq=None):
        from cake_b200.model import Context, Sessions, TextModelBase
        self.ctx = Context(cfg, sd, dtype, device=0, max_seq=max_seq or cfg.max_seq_len)
        self.model = TextModelBase.load(self.ctx)
        self.ses = Sessions(self.model, max_seq or cfg.max_seq_len)

    def run(self, rid, toks, cuts=None, end=True):
        """Feed ``toks`` as request ``rid`` in portions of the sizes ``cuts`` (cycled; None = whole) -> logits of every position."""
        out, p, i = [], 0, 0
        while p < len(toks):
            n = len(toks) - p if not cuts else min(cuts[i % len(cuts)], len(toks) - p)
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
    assert d["architecture"] == "Mafosun" and len(d["layers"]) == 5 and d["layers"][3]["mlp"] is None
    back = Config.from_hf(json.loads(json.dumps(d)))
    assert back.layers == cfg.layers and back.layer_list and back.block_kind == "mafosun" and back.embed_norm and back.tie_word_embeddings
    assert back.head_tensor_names() == ("embed", "final.norm", None) and [i for i, _ in back.run_plan()] == [0, 1, 2, 3, 4]
    p, a = back.layers[0], back.layers[1]
    assert p.type == "sink_attention" and (p.chunk, p.window, p.pool, p.v_unit, p.qk_norm, p.sink_zero, p.softcap) == (11, 0, 0, True, True, False, 0.0)
    assert p.side.type == "retention" and (p.branch_scale, p.side.branch_scale) == (0.7, 0.4) and p.side.rot.dims == 6 and not p.side.rot.interleaved
    assert (p.moe.groups, p.moe.groups_keep, p.moe.plain_weights, p.moe.act) == (3, 2, True, 0)
    assert (a.window, a.pool, a.chunk, a.sink_zero, a.softcap, a.v_unit) == (7, 3, 0, True, 5.0, False) and a.rot.interleaved
    assert a.rot.stretch == (4.0, 1.0, 4.0, 40.0) and back.layers[2].rot.stretch == () and a.dense_act == 3 and not a.pre_norms
    for path, value in ((("layers", 0, "type"), "retention"), (("layers", 1, "mixer", "kv_heads"), 3), (("layers", 1, "mixer", "rot", "dims"), 14),
                        (("layers", 1, "mlp", "kind"), "other"), (("layers", 0, "mixer", "right", "decay"), [0.5]), (("layers", 0, "mlp", "router", "top"), 9),
                        (("layers", 1, "mixer", "rot", "scaling", "high"), 0.5), (("layers", 0, "mlp", "router", "groups"), {"count": 5, "keep": 1})):
        bad = json.loads(json.dumps(d))
        node = bad
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(ValueError):
            Config.from_hf(bad)
    plainer = make_config([{"type": "attention", "mixer": {"heads": 2, "kv_heads": 2, "dim": 4, "vdim": 4, "scale": 0.5},
                            "mlp": {"kind": "moe", "router": {"experts": 3, "top": 2}, "expert": {"ff": 4}}}])
    sp = plainer.layers[0]
    assert (sp.window, sp.pool, sp.rot.dims, sp.softcap, sp.moe.groups) == (0, 0, 0, 0.0, 1)


def test_checkpoint_names_and_shapes():
    from cake_b200.loader import mafosun_block_tensors
    cfg = full_config()
    sd = make_mafosun_checkpoint(cfg, "bf16", seed=1)
    assert "head" not in sd and sd["embed.norm"].shape == (44,)
    (m0, s0), (m1, s1), (m3, _) = (mafosun_block_tensors(sd, cfg, i) for i in (0, 1, 3))
    assert m0["q"].shape == (48, 44) and m0["v"].shape == (42, 44) and m0["q_norm"].shape == (8,) and m0["o"].shape == (44, 84) and len(m0["e_gate"]) == 12
    assert s0["q"].shape == (30, 44) and s0["g"].shape == (18, 44) and s0["o"].shape == (44, 18) and s1 is None
    assert m1["k"].shape == (24, 44) and m1["post1"].shape == (44,) and m1["ff_gate"].shape == (24, 44) and "norm1" not in m1
    assert "post2" not in m3 and "router" not in m3
    bad = dict(sd)
    bad["l1.mix.k.norm"] = sd["l1.mix.k.norm"][:5]
    with pytest.raises(ValueError):
        mafosun_block_tensors(bad, cfg, 1)
    del bad["l0.mix.right.g"]
    with pytest.raises(KeyError):
        mafosun_block_tensors(bad, cfg, 0)


def test_plain_masks_and_pooled_blocks():
    w = P.window_mask(9, 3)
    assert w[8].tolist() == [False] * 6 + [True] * 3 and w[1].tolist() == [True, True] + [False] * 7
    pm = P.pool_mask(12, 4, 3, 4)       # blocks end at 2, 5, 8, 11: seen from position 6, 9, 12, ...
    assert pm[:, 0].tolist() == [False] * 6 + [True] * 6 and pm[:, 1].tolist() == [False] * 9 + [True] * 3 and not pm[:, 2].any()
    c = P.chunk_mask(7, 3)
    assert c[5].tolist() == [False, False, False, True, True, True, False] and c[6].tolist() == [False] * 6 + [True] and c[2].tolist() == [True] * 3 + [False] * 4
    k, v = torch.randn(8, 2, 3), torch.randn(8, 2, 5)
    pk, pv = P.pool_blocks(k, v, 3)
    assert pk.shape == (2, 2, 3) and torch.allclose(pk[1], (k[3] + k[4] + k[5]) / 3) and torch.allclose(pv[0], v[:3].mean(0))


def test_plain_rotations():
    f = P.frequencies({"dims": 8, "base": 200.0})
    g = P.frequencies({"dims": 8, "base": 200.0, "scaling": STRETCH})
    waves = [2 * np.pi / x for x in f]
    assert waves[0] < 10 < waves[1] < 40 < waves[2]
    s = (40 / waves[1] - 1.0) / 3.0
    assert g[0] == f[0] and abs(g[1] - ((1 - s) * f[1] / 4 + s * f[1])) < 1e-15 and g[2:] == [x / 4 for x in f[2:]]
    x = torch.randn(5, 2, 10, dtype=torch.float64)
    a, b = P.rotate(x, {"dims": 8, "base": 200.0}, True), P.rotate(x, {"dims": 8, "base": 200.0}, False)
    assert torch.allclose(a[..., 8:], x[..., 8:]) and torch.allclose(a[0], x[0]) and torch.allclose((a * a).sum(-1), (x * x).sum(-1))
    assert torch.allclose(a[3, 0, 2], x[3, 0, 2] * np.cos(3 * f[1]) - x[3, 0, 3] * np.sin(3 * f[1]))
    assert torch.allclose(b[3, 0, 5], x[3, 0, 5] * np.cos(3 * f[1]) + x[3, 0, 1] * np.sin(3 * f[1]))


def test_plain_sink_and_router():
    q, k, v = torch.zeros(2, 1, 4), torch.randn(2, 1, 4), torch.ones(2, 1, 3)
    o = P.attend(q, k, v, P.window_mask(2, 0), 1.0, 0.0, True)
    assert torch.allclose(o[0, 0], torch.full((3,), 1 / 2)) and torch.allclose(o[1, 0], torch.full((3,), 2 / 3))   # scores 0: weights 1 / (1 + keys)
    z = torch.tensor([[1.0, 0.2, 0.9, 0.8, 2.0, -9.0]])
    idx, w = P.route(z, 2, {"count": 3, "keep": 2})          # groups (0 1) (2 3) (4 5): the second is closed
    s = torch.softmax(z, -1)[0]
    assert sorted(idx[0].tolist()) == [0, 4] and torch.allclose(w.sum(), s[0] + s[4]) and float(w.sum()) < 1.0
    assert sorted(P.route(z, 3, {"count": 3, "keep": 2})[0][0].tolist()) == [0, 1, 4] and sorted(P.route(z, 3, None)[0][0].tolist()) == [0, 2, 4]


def test_plain_retention_is_a_decayed_sum():
    cfg = make_config([par(mlp=None)])
    sd = {k: v.double() for k, v in make_mafosun_checkpoint(cfg, "f32", seed=3).items()}
    m = cfg.to_hf()["layers"][0]["mixer"]["right"]
    m = dict(m, rot=None)
    h = torch.randn(6, 44, dtype=torch.float64)
    q, k, v = (P.lin(sd[f"l0.mix.right.{n}"], h).view(6, 3, -1) for n in "qkv")
    o = torch.stack([sum(float(m["decay"][hh]) ** (5 - j) * (q[5, hh] @ k[j, hh]) * 10 ** -0.5 * v[j, hh] for j in range(6)) for hh in range(3)])
    g = P.lin(sd["l0.mix.right.g"], h)[5]
    want = P.lin(sd["l0.mix.right.o"], P.rms_unit(o, 1e-5).reshape(-1) * g * torch.sigmoid(g))
    assert torch.allclose(P.retention(h, sd, "l0.mix.right.", m, 1e-5)[5], want)


# ---------------------------------------------------------------------------------------------- GPU
MECHANISMS = {
    "attention_plain": [attn(size=0, rot=0, softcap=None, mlp=None)],
    "attention_softcap": [attn(size=0, rot=0, softcap=0.5, mlp=None)],
    "attention_window_and_blocks": [attn(size=5, pool=4, rot=0, mlp=None)],
    "attention_blocks_of_one": [attn(size=4, pool=1, mlp=None)],
    "attention_block_longer_than_the_window": [attn(size=3, pool=9, mlp=None)],
    "attention_window_of_one": [attn(size=1, pool=2, mlp=None)],
    "attention_window_without_blocks": [attn(size=6, pool=0, mlp=None)],
    "attention_full_rotation": [attn(dim=12, rot=12, scaling=None, mlp=None)],
    "attention_stretched_rotation": [attn(dim=16, rot=16, base=5000.0, scaling={"factor": 8.0, "low": 0.5, "high": 3.0, "original": 30}, mlp=None)],
    "attention_every_head_its_keys": [attn(heads=3, kv_heads=3, mlp=None)],
    "attention_one_key_head": [attn(heads=5, kv_heads=1, dim=20, vdim=36, rot=6, mlp=None)],
    "attention_wide_heads": [attn(heads=2, kv_heads=1, dim=72, vdim=136, rot=40, mlp=None)],
    "attention_head_of_300": [attn(heads=1, kv_heads=1, dim=300, vdim=20, rot=300, mlp=None)],
    "parallel": [par(mlp=None)],
    "parallel_left_only": [par(rs=0.0, mlp=None)],
    "parallel_right_only": [par(ls=0.0, mlp=None)],
    "parallel_scales_of_one": [par(ls=1.0, rs=1.0, mlp=None)],
    "parallel_no_chunks_no_rotation": [par(size=0, rot=0, mlp=None)],
    "parallel_chunks_of_one": [par(size=1, mlp=None)],
    "parallel_one_head_each": [par(heads=1, kv_heads=1, dim=5, vdim=7, rheads=1, rdim=6, rvdim=3, rot=2, decay=[0.75], mlp=None)],
    "parallel_register_state": [par(rheads=2, rdim=32, rvdim=32, rot=32, mlp=None)],
    "parallel_register_state_wide": [par(rheads=2, rdim=48, rvdim=64, rot=16, decay=[1.0, 0.9], mlp=None)],
    "parallel_state_of_80_by_40": [par(rheads=1, rdim=80, rvdim=40, rot=80, decay=[0.96], mlp=None)],
    "dense": [attn(size=0, rot=0, softcap=None, mlp=dense(56))],
    "experts": [attn(mlp=moe())],
    "experts_one_group": [attn(mlp=moe(groups=1, keep=1))],
    "experts_every_group_kept": [attn(mlp=moe(groups=4, keep=4))],
    "experts_top_one": [attn(mlp=moe(experts=6, top=1, groups=3, keep=1))],
    "experts_all_of_a_group": [attn(mlp=moe(experts=8, top=4, groups=2, keep=1))],
    "experts_of_one_each": [attn(mlp=moe(experts=6, top=2, groups=6, keep=2))],
    "experts_many": [attn(mlp=moe(experts=80, top=7, ff=8, groups=40, keep=5))],
    "experts_one": [attn(mlp=moe(experts=1, top=1, ff=20, groups=1, keep=1))],
}


@pytest.mark.gpu
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_each_mechanism_alone(name):
    cfg = make_config(MECHANISMS[name])
    sd = make_mafosun_checkpoint(cfg, "f32", seed=sum(map(ord, name)) % 1000)
    toks = tokens(41, cfg.vocab_size, seed=3)
    want = plain(cfg, sd, toks)
    r = Runner(cfg, sd, "f32")
    try:
        close(r.run("a", toks), want, "f32", "whole")
        close(r.run("b", toks, cuts=[1]), want, "f32", "token by token")
        close(r.run("c", toks, cuts=[2, 5, 3]), want, "f32", "portions")
    finally:
        r.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["f32", "f16"])
def test_residual_after_every_layer(dtype):
    from cake_b200.capi import check, lib, ptr
    cfg = full_config()
    sd = make_mafosun_checkpoint(cfg, dtype, seed=5)
    toks = tokens(29, cfg.vocab_size, seed=4)
    streams = []
    plain(cfg, sd, toks, streams)
    r = Runner(cfg, sd, dtype)
    try:
        ctx, model = r.ctx, r.model
        for lo, hi in ((0, 17), (17, 29)):     # two portions: the second reads cache rows and state of the first in every layer
            ids = np.ascontiguousarray([toks[lo:hi]], dtype=np.uint32)
            x = ctx.empty(1, hi - lo, cfg.hidden_size, dtype=torch.float32)
            check(lib().cake_b200_embed(ctx.h, ids.ctypes.data_as(ctypes.POINTER(ctypes.c_uint32)), 1, hi - lo, ptr(x)))
            for j, blk in enumerate(model.blocks):
                x = blk.forward_batch(x, [(blk.layer_name(), lo, j)], ctx, blocks=[blk])
                ctx.sync()
                want = streams[j][lo:hi].numpy()
                d = np.abs(x[0].cpu().numpy() - want).max(-1)
                bar = (2e-4 if dtype == "f32" else 3e-2) * max(1.0, np.abs(want).max())
                assert (d.max() if dtype == "f32" else np.quantile(d, 0.9)) < bar, f"layer {j}, tokens {lo}..{hi}: {d.max():.3g}"
        assert len(model.blocks) == len(streams) == 5
    finally:
        r.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["f32", "bf16", "f16"])
def test_schedules_agree_with_the_plain_model(dtype):
    cfg = full_config()
    sd = make_mafosun_checkpoint(cfg, dtype, seed=11)
    toks = tokens(83, cfg.vocab_size, seed=5)
    want = plain(cfg, sd, toks)
    bar = None
    if dtype != "f32":
        to = torch.bfloat16 if dtype == "bf16" else torch.float16
        bar = max(TOL[dtype], 2 * float(np.quantile(errors(plain_with_rounded_products(cfg, sd, toks, to), want), 0.95)))
    r = Runner(cfg, sd, dtype)
    try:
        whole = r.run("w", toks)
        close(whole, want, dtype, "whole", bar)
        for cuts in ([1], [2], [2, 3, 5], [17], [64, 1], [1, 40, 2]):
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
    sd = make_mafosun_checkpoint(cfg, "f32", seed=21)
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
        close(r.run("c", c, cuts=[9, 1]), wc, "f32", "a longer request in a used slot")    # rows, blocks and states of the old request lie there
        close(r.run("d", b, cuts=[4]), wb, "f32", "a shorter request in a used slot")
        close(r.run("e", a), wa, "f32", "whole in a used slot")
        assert len(r.ses.free) == 2 and not r.ses.live
    finally:
        r.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_batch_rows_against_each_alone(dtype):
    cfg = full_config()
    sd = make_mafosun_checkpoint(cfg, dtype, seed=31)
    rows = [tokens(40, cfg.vocab_size, seed=20 + i) for i in range(3)]
    want = [plain(cfg, sd, t) for t in rows]
    r = Runner(cfg, sd, dtype)
    try:
        got = r.rows(rows, (23, 1, 1, 15), 64)
        for i in range(3):
            bar = None if dtype == "f32" else max(TOL[dtype], 2 * float(np.quantile(errors(plain_with_rounded_products(cfg, sd, rows[i]), want[i]), 0.95)))
            close(got[i], want[i], dtype, f"batch row {i}", bar)
    finally:
        r.close()


def show_faults(cfg, sd, toks, want, names, bar):
    for f in names:
        e = errors(plain(cfg, sd, toks, fault=f), want)
        assert e.max() > bar, f"{f} would not show: {e.max():.3g}"


@pytest.mark.gpu
@pytest.mark.parametrize("kind", ["attention", "parallel"])
def test_edges_of_windows_blocks_and_chunks(kind):
    """Sharp scores, so that single keys carry a row.  A window one position longer or shorter, blocks that come one position early or
    late or not at all, no sink, a chunk one position longer, no chunks: each changes the plain model's logits by many tolerances;
    the framework agrees with the right one in a whole prompt, in portions cut at and around every edge, and token by token."""
    if kind == "attention":
        layers = [attn(size=11, pool=4, scale=1.5, softcap=20.0, mlp=None), attn(heads=2, kv_heads=1, size=6, pool=5, scale=1.2, rot=4, mlp=dense())]
        faults = ("window+1", "window-1", "pool early", "pool late", "no pool", "no sink")
    else:
        layers = [par(size=11, scale=1.5, mlp=None), par(heads=2, kv_heads=1, size=6, scale=1.2, mlp=dense())]
        faults = ("chunk+1", "no chunk")
    cfg = make_config(layers)
    sd = make_mafosun_checkpoint(cfg, "f32", seed=41)
    toks = tokens(90, cfg.vocab_size, seed=9)
    want = plain(cfg, sd, toks)
    show_faults(cfg, sd, toks, want, faults, 50 * TOL["f32"])
    r = Runner(cfg, sd, "f32")
    try:
        close(r.run("w", toks), want, "f32", "whole")
        for cuts in ([11], [10], [12], [4], [5], [6, 5], [1], [3] + [1] * 12, [40, 2]):
            close(r.run("c", toks, cuts=cuts), want, "f32", f"portions {cuts}")
    finally:
        r.close()
    sb = {k: v.to(torch.bfloat16) for k, v in sd.items()}
    wb = plain(cfg, sb, toks)
    bar = max(TOL["bf16"], 2 * float(np.quantile(errors(plain_with_rounded_products(cfg, sb, toks), wb), 0.95)))
    rb = Runner(cfg, sb, "bf16")
    try:
        close(rb.run("w", toks), wb, "bf16", "whole, bf16", bar)
        close(rb.run("c", toks, cuts=[30, 1]), wb, "bf16", "decoded, bf16", bar)
    finally:
        rb.close()


@pytest.mark.gpu
def test_group_limit_and_plain_weights():
    cfg = make_config([attn(mlp=moe(experts=12, top=3, groups=4, keep=2)), par(mlp=moe(experts=9, top=2, groups=3, keep=1))])
    sd = make_mafosun_checkpoint(cfg, "f32", seed=44)
    toks = tokens(60, cfg.vocab_size, seed=19)
    want = plain(cfg, sd, toks)
    show_faults(cfg, sd, toks, want, ("no groups",), 50 * TOL["f32"])
    big = dict(sd)      # the output norm hides a common factor of the weights unless the sum is small beside eps
    for i in (0, 1):
        for j in range(12):
            if f"l{i}.mlp.e{j}.down" in big:
                big[f"l{i}.mlp.e{j}.down"] = sd[f"l{i}.mlp.e{j}.down"] * 1e-3
    wbig = plain(cfg, big, toks)
    show_faults(cfg, big, toks, wbig, ("renormalised",), 20 * TOL["f32"])
    for weights, w in ((sd, want), (big, wbig)):
        r = Runner(cfg, weights, "f32")
        try:
            close(r.run("w", toks), w, "f32", "whole")
            close(r.run("c", toks, cuts=[9, 1, 1]), w, "f32", "portions")
        finally:
            r.close()


def f16_case(layers, width, vocab, n, seed, faults, start=0):
    """A configuration in f16 (where rounding is small) with flat scores, so that every edge fault moves most positions: -> (cfg, sd,
    toks, want, bar) after showing that each fault would be seen."""
    cfg = make_config(layers, width=width, vocab=vocab)
    sd = make_mafosun_checkpoint(cfg, "f16", seed=seed)
    toks = tokens(n, vocab, seed=13)
    want = plain(cfg, sd, toks)
    bar = max(4 * float(np.quantile(errors(plain_with_rounded_products(cfg, sd, toks, torch.float16), want), 0.95)), 3e-3)
    for f in faults:
        e = errors(plain(cfg, sd, toks, fault=f)[start:], want[start:])
        assert np.quantile(e, 0.5) > 2 * bar or e.max() > 12 * bar, f"{f} would not show: {np.quantile(e, 0.5):.3g}, {e.max():.3g} against {bar:.3g}"
    return cfg, sd, toks, want, bar


@pytest.mark.gpu
def test_key_size_128_portions_on_the_tensor_core_attention():
    """Key and value size 128 in 16-bit D: portions of 64 rows and more take the tensor-core attention (the tiles of the pooled blocks
    ahead of the window's, chunks, the soft cap, the zero sink, both mixers' heads side by side in one output row), shorter ones
    the other kernels.  A window, block or chunk that is one off moves the plain model's logits by several bars."""
    layers = [attn(heads=2, kv_heads=1, dim=128, vdim=128, size=9, pool=2, scale=0.02, softcap=30.0, rot=64, base=1000.0, scaling=None, mlp=None),
              par(heads=2, kv_heads=2, dim=128, vdim=128, size=70, scale=0.05, rheads=2, rdim=32, rvdim=64, rot=32, mlp=dense(128)),
              attn(heads=4, kv_heads=2, dim=128, vdim=128, size=70, pool=3, scale=0.02, softcap=30.0, rot=128, mlp=None)]
    # layer 0 and layer 1 see few keys per row, so one key more or less shows; layer 2 walks several tiles of blocks and of its window
    cfg, sd, toks, want, bar = f16_case(layers, 128, 96, 700, 47, ("window+1", "window-1", "pool early", "pool late", "no pool", "no sink", "chunk+1", "no chunk"))
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
    layers = [attn(heads=2, kv_heads=1, dim=24, vdim=40, size=9, pool=2, scale=0.05, softcap=30.0, rot=16, base=1000.0, scaling=None, mlp=None),
              par(heads=4, kv_heads=2, dim=64, vdim=112, size=66, scale=0.05, rheads=1, rdim=64, rvdim=32, rot=64, decay=[0.98], mlp=dense(64)),
              attn(heads=3, kv_heads=3, dim=96, vdim=96, size=65, pool=4, scale=0.05, softcap=30.0, rot=96, mlp=moe(8, 2, 64, 2, 1))]
    cfg, sd, toks, want, bar = f16_case(layers, 128, 128, 330, 48, ("window+1", "window-1", "pool early", "pool late", "no pool", "no sink", "no chunk"))
    r = Runner(cfg, sd, "f16")
    try:
        whole = r.run("w", toks)
        close(whole, want, "f16", "whole", bar)
        for cuts in ([200, 130], [64, 66], [37], [150, 1, 1, 1, 100, 2]):
            close(r.run("c", toks, cuts=cuts), want, "f16", f"portions {cuts}", bar)
    finally:
        r.close()


@pytest.mark.gpu
def test_a_far_block_carries_weight():
    """Queries of one token match the keys of another that fills one early block: 400 positions back it still decides the row, through
    its mean.  Without that block's token the plain model's logits move by many tolerances; whole, in portions and decoded (over more
    than 256 visible keys the split-key kernels run)."""
    cfg = make_config([attn(heads=2, kv_heads=2, dim=16, vdim=16, size=40, pool=2, scale=1.0, softcap=60.0, rot=4, base=1e6, scaling=None, mlp=None),
                       par(size=300, scale=1.5, mlp=None)])
    sd = make_mafosun_checkpoint(cfg, "f32", seed=43)
    ask, answer = 7, 9
    sd["embed.norm"] = torch.ones_like(sd["embed.norm"])
    e = P.rms_unit(sd["embed"], 1e-5)
    u = (e[ask] - e[answer]) / (e[ask] - e[answer]).norm()
    sd["l0.mix.q"] = sd["l0.mix.k"] @ (torch.eye(44) - 2 * u[:, None] * u[None, :])     # swaps the two embeddings, then looks for keys
    sd["l0.mix.q.norm"] = sd["l0.mix.k.norm"].clone()
    toks = [t if t not in (ask, answer) else 8 for t in tokens(460, cfg.vocab_size, seed=10)]
    toks[20] = toks[21] = answer
    toks[455] = toks[456] = ask
    want = plain(cfg, sd, toks)
    other = list(toks)
    other[20] = other[21] = 3
    assert errors(plain(cfg, sd, other), want)[[455, 456]].min() > 50 * TOL["f32"]      # the far block decides these rows
    show_faults(cfg, sd, toks, want, ("no pool", "no chunk"), 50 * TOL["f32"])
    r = Runner(cfg, sd, "f32")
    try:
        close(r.run("w", toks), want, "f32", "whole")
        close(r.run("c", toks, cuts=[129, 127, 2, 1]), want, "f32", "portions")
        close(r.run("d", toks, cuts=[400] + [1] * 60), want, "f32", "decoded")
    finally:
        r.close()
    sb = {k: v.to(torch.bfloat16) for k, v in sd.items()}
    wb = plain(cfg, sb, toks)
    bar = max(TOL["bf16"], 2 * float(np.quantile(errors(plain_with_rounded_products(cfg, sb, toks), wb), 0.95)))
    rb = Runner(cfg, sb, "bf16")
    try:
        close(rb.run("d", toks, cuts=[400] + [1] * 60), wb, "bf16", "decoded, bf16", bar)
    finally:
        rb.close()


@pytest.mark.gpu
def test_long_decoding_past_every_window_and_chunk():
    cfg = full_config()
    sd = make_mafosun_checkpoint(cfg, "f32", seed=45)
    toks = tokens(230, cfg.vocab_size, seed=11)
    want = plain(cfg, sd, toks)
    r = Runner(cfg, sd, "f32")
    try:
        close(r.run("d", toks, cuts=[10] + [1] * 220), want, "f32", "a short prompt then long decoding")
    finally:
        r.close()


@pytest.mark.gpu
def test_a_cache_that_the_request_fills_to_the_last_row():
    """The capacity is no multiple of the block size: the last incomplete block has no row of its own."""
    cfg = make_config([attn(size=5, pool=4), par(size=9)])
    sd = make_mafosun_checkpoint(cfg, "f32", seed=46)
    toks = tokens(31, cfg.vocab_size, seed=15)
    want = plain(cfg, sd, toks)
    r = Runner(cfg, sd, "f32", max_seq=31)
    try:
        close(r.run("w", toks), want, "f32", "whole")
        close(r.run("c", toks, cuts=[7, 1]), want, "f32", "portions")
        from cake_b200.capi import CakeB200Error
        r.run("full", toks, end=False)
        with pytest.raises(CakeB200Error):
            r.ses.step("full", [1], want=[0])
        r.ses.end("full")
    finally:
        r.close()
    short = make_config([attn(size=5, pool=64)])       # blocks longer than the cache
    s2 = make_mafosun_checkpoint(short, "f32", seed=47)
    r = Runner(short, s2, "f32", max_seq=20)
    try:
        close(r.run("w", toks[:20], cuts=[3]), plain(short, s2, toks[:20]), "f32", "blocks longer than the cache")
    finally:
        r.close()


@pytest.mark.gpu
def test_other_sizes_and_tensor_core_shapes():
    """Sizes whose projections and experts take the tensor-core kernels (multiples of 128 / 64) next to ones that do not; long
    portions and decoding; against the plain model and whole against portions."""
    layers = [attn(heads=4, kv_heads=2, dim=64, vdim=64, size=96, pool=8, scale=0.3, softcap=15.0, rot=32, base=1000.0, mlp=dense(128)),
              par(heads=4, kv_heads=1, dim=32, vdim=64, size=70, scale=0.3, rheads=4, rdim=32, rvdim=32, rot=32, mlp=moe(6, 2, 64, 3, 2)),
              attn(heads=2, kv_heads=1, dim=128, vdim=128, size=40, pool=16, scale=0.2, rot=64, scaling=None, mlp=moe(8, 3, 128, 2, 1)),
              par(heads=3, kv_heads=3, dim=24, vdim=40, size=33, scale=0.4, rheads=2, rdim=24, rvdim=20, rot=10, mlp=dense(72))]
    cfg = make_config(layers, width=128, vocab=256)
    for dtype in ("bf16", "f32"):
        sd = make_mafosun_checkpoint(cfg, dtype, seed=51)
        toks = tokens(300, cfg.vocab_size, seed=12)
        want = plain(cfg, sd, toks)
        # 16 bits: twice what rounding the products alone does to this configuration (its routed layers flip experts)
        bar = 2 * float(np.quantile(errors(plain_with_rounded_products(cfg, sd, toks), want), 0.95)) if dtype == "bf16" else None
        r = Runner(cfg, sd, dtype)
        try:
            whole = r.run("w", toks)
            close(whole, want, dtype, "whole", bar)
            close(r.run("c", toks, cuts=[133, 2, 1, 150, 1]), want, dtype, "portions", bar)
            close(r.run("d", toks, cuts=[260] + [1] * 40), want, dtype, "decoded", bar)
            if dtype == "bf16":   # the schedules agree with each other more closely than with the exact model
                close(r.run("c", toks, cuts=[133, 2, 1, 150, 1]), whole, dtype, "portions against whole", bar)
        finally:
            r.close()
    # without routers no position has an excuse: all of them within twice the worst that rounding the products causes
    for L in layers:
        L["mlp"] = dense(64)
    cfg = make_config(layers, width=128, vocab=256)
    sd = make_mafosun_checkpoint(cfg, "bf16", seed=53)
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
    """Parts that are not built together are refused at load with a message, not computed wrongly."""
    from cake_b200.capi import CakeB200Error
    cfg = make_config([attn()])
    sd = make_mafosun_checkpoint(cfg, "f32", seed=52)
    for edit in (dict(chunk=4), dict(keep_first=2), dict(qk_unit=True), dict(softcap=-1.0)):
        bad = copy.deepcopy(cfg)
        for k, v in edit.items():
            setattr(bad.layers[0], k, v)
        with pytest.raises(CakeB200Error):
            Runner(bad, sd, "f32")


@pytest.mark.gpu
def test_greedy_generation_through_master():
    from cake_b200.model import Context, Master, TextModelBase
    cfg = full_config()
    sd = make_mafosun_checkpoint(cfg, "f32", seed=61)
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
    sd = make_mafosun_checkpoint(cfg, "bf16", seed=81)
    model_dir, out_dir = str(tmp_path / "model"), str(tmp_path / "out")
    save_checkpoint(model_dir, cfg, sd)
    back, vb = open_model(model_dir)
    assert set(vb.keys()) == set(sd.keys()) and back.block_kind == "mafosun"
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
