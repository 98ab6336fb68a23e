"""The Rufisun design on the GPU against the plain implementation of plain_rufisun.py: each mechanism alone (the norm by tanh, the
growing queries, attention at the edges of its window and of its kept first tokens, sinks and caps, latent attention with a
stretched rotation, the state space in its dual form, weights on the experts' inputs, the products' epilogues), then whole models
under every way of cutting the work and greedy generation through the engine's entry point, the replay program and the command
line.  Configurations and weights are made here."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_rufisun as plain
from helpers import MEAN_TOL, TOL, Replayer
from test_lutodra_gpu import DT, LENGTHS, SCHEDULE, dev, run_mixer, stored
from test_rufisun_config import att, cap, config, dense, lat, moe, par, ssd

pytestmark = pytest.mark.gpu

# every branch: head and value sizes that differ, groups of query heads, windows shorter and longer than the kept tokens, none kept,
# no window, latent rows with and without stretching, groups of the state space, one norm part and several, convolutions of one tap
# and more, dense and routed feed-forwards with and without a shared expert, layers without a feed-forward
CFG_A = config([att(6, 2, 12, 20, scale=0.4, bias_max=50, mask=(24, 5), mlp=dense(96)),
                lat(3, 10, 6, 14, 20, 24, scale=0.3, mlp=moe(24, 5, 2, shared=40)),
                par(cap(4, 2, 16, 8, scale=0.35), ssd(6, 8, 12, groups=3, norm_groups=2), mlp=moe(40, 8, 1, shared=24)),
                att(4, 4, 8, 8, scale=0.5, bias_max=33.5, mask=(9, 14), mlp=moe(16, 3, 3))], width=64, vocab=200)
CFG_B = config([par(cap(3, 3, 10, 14, softcap=2.5, q_temp=(1.1, 7)), ssd(5, 7, 9, conv=5, norm_groups=5)), lat(2, 24, 2, 24, 33, 7, base=50.0, mlp=dense(50)),
                att(5, 1, 8, 12, mask=(17, 1), bias_max=200, mlp=moe(20, 6, 2)), att(2, 2, 24, 24, mask=(40, 0)),
                lat(4, 8, 12, 6, 12, 16, scaling=None)], width=72, vocab=301, eps=1e-6)
CFG_C = config([att(8, 2, 64, 64, scale=0.15, bias_max=90, mask=(37, 6), mlp=dense(80)),
                par(cap(4, 4, 128, 128, scale=0.09, softcap=9.0), ssd(4, 32, 48, groups=2, norm_groups=4), mlp=moe(48, 6, 2, shared=56)),
                lat(4, 32, 16, 24, 48, 32, scale=0.2, mlp=moe(24, 4, 1, shared=32)),
                att(4, 4, 128, 128, scale=0.1, bias_max=150, mask=(70, 130), mlp=dense(64)),
                par(cap(6, 2, 64, 64, scale=0.125, q_temp=(0.2, 50)), ssd(8, 16, 16, norm_groups=1), mlp=dense(40))], width=88, vocab=264)
CONFIGS = {"A": (CFG_A, 16), "B": (CFG_B, 32), "C": (CFG_C, 16)}
SHARP = {"float32": 1.7, "bfloat16": 1.0}


def compare(got, want, dtype, what="", slack=None):
    """Rows of logits against the plain implementation's: every row within TOL of the largest logit, in bfloat16 plus twice what
    perturbations of bfloat16's size cause in the plain implementation at that row (plain.rounding_error); the mean error within
    MEAN_TOL over the rows, with the same addition."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape and np.isfinite(got).all(), what
    scale = np.abs(want).max()
    extra = np.zeros(len(want)) if dtype == "float32" or slack is None else 2 * np.asarray(slack) / scale
    rows = np.abs(got - want).max(axis=1) / scale
    bad = rows > TOL[dtype] + extra
    assert not bad.any(), f"{what}: {bad.sum()} of {len(rows)} rows too far, worst {rows.max():.3e} at row {int(rows.argmax())}, slack there {extra[rows.argmax()]:.3e}"
    mean = np.abs(got - want).mean() / scale
    assert mean <= MEAN_TOL[dtype] + extra.mean(), f"{what}: mean error {mean:.3e}"


def slack_of(cfg, w, ids, dtype):
    return None if dtype == "float32" else plain.rounding_error(cfg, w, ids, runs=4)


def make_weights(cfg, seed, dtype):
    # bfloat16 rounds the routers' inputs: there constant coordinates decide who is chosen
    w = plain.random_weights(cfg, seed, sharp=SHARP[dtype], decisive_routing=dtype == "bfloat16")
    return plain.round_to_bf16(w) if dtype == "bfloat16" else w


def ids_of(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()


def build(tmp_path, name, dtype, num_pages, seed=1, max_seqs=4, graphs=False, cfg_page=None):
    from vllm_cpp_b200 import EngineConfig
    from vllm_cpp_b200.engine import factory
    cfg, page = cfg_page or CONFIGS[name]
    weights = make_weights(cfg, seed, dtype)
    folder = str(tmp_path / f"rufisun_{name}_{dtype}")
    plain.write_model_folder(folder, cfg, weights, store="BF16" if dtype == "bfloat16" else "F32")
    ecfg = EngineConfig(model_path=folder, dtype=dtype, block_size=page, num_gpu_blocks=num_pages, max_num_seqs=max_seqs,
                        max_model_len=num_pages * page, max_num_batched_tokens=1024, use_cuda_graphs=graphs)
    model, cache, runner = factory.build(ecfg)
    return cfg, weights, folder, cache, runner


def part_of(layer, width, dtype, eps=1e-5, slot="mixer"):
    """The engine's part for one layer of a configuration."""
    from vllm_cpp_b200.config.registry import resolve_architecture
    from vllm_cpp_b200.parts import model  # noqa: F401  (registers the parts)
    from vllm_cpp_b200.parts.base import FEED_FORWARDS, MIXERS, build_part
    _, spec = resolve_architecture(config([layer], width=width, eps=eps))
    table = {"mixer": MIXERS, "feed_forward": FEED_FORWARDS}[slot]
    return build_part(table, slot, spec.layers[0].parts[slot], dtype=DT[dtype], device="cuda")


def part_weights(w, p, dtype, part):
    return {n: dev(np.asarray(w[p + n], dtype=np.float32), torch.float32 if ps.role != "matrix" else DT[dtype])
            for n, ps in part.param_specs().items()}


def rounded(w, dtype):
    return plain.round_to_bf16(w) if dtype == "bfloat16" else w


# ------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,n", [(72, 5), (77, 3), (320, 9), (2504, 2), (4096, 3)])
def test_norm_by_tanh(dtype, width, n):
    """With and without a pending addition, gathered rows, two results joined; the stream stays float."""
    from vllm_cpp_b200.csrc import ops
    rng = np.random.default_rng(width)
    x = (3 * rng.standard_normal((n, width))).astype(np.float32)
    a, b = stored(rng.standard_normal((n, width)), dtype), stored(rng.standard_normal((n, width)), dtype)
    w = {"n": rng.standard_normal(width).astype(np.float32), "n.b": rng.standard_normal(width).astype(np.float32), "n.alpha": np.float32(0.37)}
    args = (dev(np.array([0.37], dtype=np.float32)), dev(w["n"]), dev(w["n.b"]))
    tol = 2e-6 if dtype == "float32" else 5e-3
    out = torch.empty((n, width), dtype=DT[dtype], device="cuda")
    for delta, delta2, sums in ((None, None, x), (a, None, x + 0.5 * a), (a, b, x + 0.5 * a - 1.5 * b)):
        dx = dev(x)
        ops.add_tanh_norm(dx, None if delta is None else dev(delta, DT[dtype]), *args, out, None, 0.5, None if delta2 is None else dev(delta2, DT[dtype]), -1.5)
        assert np.abs(dx.cpu().numpy() - sums).max() <= 1e-5
        want = plain.tanh_norm(sums.astype(np.float64), w, "n")
        assert np.abs(out.float().cpu().numpy() - want).max() <= tol * np.abs(want).max()
    rows = np.array([n - 1, 0, n - 1], dtype=np.int32)
    some = torch.empty((3, width), dtype=DT[dtype], device="cuda")
    dx = dev(x)
    ops.add_tanh_norm(dx, dev(a, DT[dtype]), *args, some, dev(rows), 1.0)
    want = plain.tanh_norm(x.astype(np.float64) + a, w, "n")[rows]
    assert np.abs(some.float().cpu().numpy() - want).max() <= tol * np.abs(want).max() and (dx.cpu().numpy() == x).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("act", ["relu_squared", "gelu"])
@pytest.mark.parametrize("width,ff", [(64, 96), (72, 50), (320, 384), (33, 21)])
def test_feed_forward_without_a_gate(dtype, act, width, ff):
    """Few and many tokens: the activation in the product's epilogue (bfloat16, few tokens) and as a kernel after it."""
    from vllm_cpp_b200.csrc import ops
    from vllm_cpp_b200.parts.base import Workspace
    from vllm_cpp_b200.parts.mlp import TwoLayerMLP
    rng = np.random.default_rng(width)
    w = rounded({"up": 2 * rng.standard_normal((ff, width)) / np.sqrt(width), "down": rng.standard_normal((width, ff)) / np.sqrt(ff)}, dtype)
    part = TwoLayerMLP(width, ff, act, DT[dtype], "cuda")
    part.load_params({k: dev(v.astype(np.float32), DT[dtype]) for k, v in w.items()})
    ops.forget_choices(ff, width)
    ops.forget_choices(width, ff)
    for n in (1, 9, 40, 100, 200):
        h = stored(rng.standard_normal((n, width)), dtype)
        out = torch.empty((n, width), dtype=DT[dtype], device="cuda")
        part.forward(dev(h, DT[dtype]), out, None, Workspace("cuda"))
        want = (plain.dense_ff if act == "relu_squared" else plain.expert_ff)(h, w, "")
        assert np.abs(out.float().cpu().numpy() - want).max() <= (2e-5 if dtype == "float32" else 2e-2) * np.abs(want).max(), n
    ops.check_status()


@pytest.mark.parametrize("n", [1, 7, 16, 20, 50, 100, 128])
@pytest.mark.parametrize("features,k,tiled", [(320, 96, False), (88, 64, True), (1024, 512, True)])
def test_a_product_that_ends_a_branch_before_a_norm_by_tanh(n, features, k, tiled):
    """residual += x W^T and the finished norm out of one kernel, and an activation out of one, beside the operations one by one."""
    from vllm_cpp_b200.csrc import ops
    rng = np.random.default_rng(n + features)
    x, w = stored(rng.standard_normal((n, k)), "bfloat16"), stored(rng.standard_normal((features, k)) / np.sqrt(k), "bfloat16")
    res = rng.standard_normal((n, features)).astype(np.float32)
    g, b, alpha = rng.standard_normal(features).astype(np.float32), rng.standard_normal(features).astype(np.float32), np.array([0.8], dtype=np.float32)
    dw, dx, dr = dev(w, torch.bfloat16), dev(x, torch.bfloat16), dev(res)
    if tiled:
        ops.tile_weights(dw)
    out = torch.empty((n, features), dtype=torch.bfloat16, device="cuda")
    ops.gemm_bf16_tcgen05(dx, dw, out, fuse=ops.ResidualTanhNorm(dr, dev(alpha), dev(g), dev(b)))
    ops.check_status()
    new = res + x @ w.T
    assert np.abs(dr.cpu().numpy() - new).max() <= 1e-4
    want = np.tanh(alpha[0] * new) * g + b
    assert np.abs(out.float().cpu().numpy() - want).max() <= 5e-3 * np.abs(want).max()
    for act, f in (("relu_squared", lambda z: np.maximum(z, 0) ** 2), ("gelu", plain.gelu)):
        ops.gemm_bf16_tcgen05(dx, dw, out, act=act)
        want = f(x @ w.T)
        assert np.abs(out.float().cpu().numpy() - want).max() <= 5e-3 * np.abs(want).max(), act
    ops.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 12, 20), (2, 2, 64, 64), (3, 1, 16, 8)])
def test_queries_grow_with_their_position(dtype, H, G, dk, dv):
    """At the steps of the quotient, and only the queries."""
    from vllm_cpp_b200.csrc import ops
    rng = np.random.default_rng(H)
    pos = np.array([0, 1, 5, 6, 7, 12, 13, 14, 200, 1000003], dtype=np.int32)
    n, C = len(pos), H * dk + G * (dk + dv)
    proj = stored(rng.standard_normal((n, C)), dtype)
    q = torch.empty((n, H * dk), dtype=DT[dtype], device="cuda")
    page, row = 16, max(dk, dv)
    pages = torch.zeros((2, 2 * G * page * row), dtype=DT[dtype], device="cuda")
    ops.qk_norm_cache_write(dev(proj, DT[dtype]), 0, H * dk, (H + G) * dk, None, None, q, pages, dev(pos), dev(np.zeros(n, dtype=np.int32)),
                            dev(np.zeros((1, 70000), dtype=np.int32)), num_heads=H, num_kv_heads=G, head_dim=dk, v_head_dim=dv, row=row, page_size=page,
                            eps=1e-5, write_kv=False, temperature=(0.6, 7))
    want = proj[:, :H * dk] * plain.query_temperature(pos.astype(np.float64), 0.6, 7)[:, None]
    assert np.abs(q.float().cpu().numpy() - want).max() <= (2e-6 if dtype == "float32" else 5e-3) * np.abs(want).max()
    t = plain.query_temperature(pos.astype(np.float64), 0.6, 7)
    assert t[0] == t[2] == 1.0 and t[3] == t[5] > 1.0 and t[6] > t[5]          # positions 5, 6 and 12, 13 lie on either side of a step


def lone_keys(dtype, H, G, dk, dv, page, marks, n=190, width=24, look_scale=3.0):
    """A mixer's weights and inputs in which a few tokens' keys are what every query looks for."""
    rng = np.random.default_rng(H * 100 + dk)
    look = rng.standard_normal(dk)
    look /= np.linalg.norm(look)
    w = {"q": np.zeros((H * dk, width)), "k": np.zeros((G * dk, width)), "v": rng.standard_normal((G * dv, width)) / np.sqrt(width),
         "o": rng.standard_normal((width, H * dv)) / np.sqrt(H * dv), "g": rng.standard_normal((H * dv, width)) / np.sqrt(width),
         "sink": np.linspace(4.0, 5.5, H), "rel": 0.5 * rng.standard_normal((12, H))}
    w["q"][:, 1] = np.tile(look * look_scale, H)
    w["k"][:, 0] = np.tile(look * 2.0, G)
    x = rng.standard_normal((n, width))
    x[:, 0], x[:, 1] = 0.0, 1.0
    for m in marks:
        x[m, 0] = 1.0 + 0.1 * (m % 3)
    return rounded(w, dtype), stored(x, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,size,keep,page", [(4, 2, 16, 24, 20, 6, 8), (2, 1, 8, 8, 5, 13, 16), (3, 3, 12, 4, 1, 1, 16), (8, 2, 64, 64, 37, 6, 16),
                                                      (4, 1, 128, 128, 64, 16, 16), (4, 4, 64, 64, 130, 7, 8), (2, 2, 64, 64, 24, 0, 8),
                                                      (16, 1, 64, 64, 9, 70, 32), (6, 2, 128, 128, 3, 129, 16)])
@pytest.mark.parametrize("cut", ["whole", "portions", "decode"])
def test_attention_just_inside_and_just_outside_its_window_and_kept_tokens(dtype, H, G, dk, dv, size, keep, page, cut):
    """Tokens whose keys stand out, in the kept tokens' last places, just after them, at page borders and in the middle.  The engine
    agrees with the plain rule at every position, and every rule that is one off is far from it at some position."""
    width, n = 24, 190
    marks = {0, max(keep - 1, 0), keep, page - 1, 60, 61 + size % 50}
    w, x = lone_keys(dtype, H, G, dk, dv, page, marks)
    layer = att(H, G, dk, dv, scale=1.0, bias_max=50, mask=(size, keep))
    part = part_of(layer, width, dtype)
    part.load_params(part_weights(w, "", dtype, part))
    schedule = {"whole": [[("a", n)]], "portions": [[("a", t)] for t in (2, 30, 3, 64, 17, 2, 40, 32)],
                "decode": [[("a", 41)]] + [[("a", 1)] for _ in range(n - 41)]}[cut]
    got, _ = run_mixer(part, {"a": x}, schedule, page=page, pages=30, max_len=240, width_out=width)

    def rule(size, keep, sink=w["sink"], rel=w["rel"]):
        q, k, v = ((x @ w[t].T).reshape(n, -1, d) for t, d in (("q", dk), ("k", dk), ("v", dv)))
        o = plain.attention_core(q, k, v, 1.0, sink, size, keep, rel, 50)
        return (o.reshape(n, -1) * plain.sigmoid(x @ w["g"].T)) @ w["o"].T

    want = rule(size, keep)
    assert np.abs(got["a"] - want).max() <= (3e-5 if dtype == "float32" else 2e-2) * np.abs(want).max()
    if cut == "whole" and dtype == "float32":
        wrong = [rule(size + 1, keep), rule(size, keep + 1), rule(size, keep, np.full(H, -60.0)), rule(size, keep, rel=np.roll(w["rel"], 1, axis=0))]
        wrong += [rule(size - 1, keep)] if size > 1 else []
        wrong += [rule(size, keep - 1), rule(size, 0)] if keep else []
        for i, other in enumerate(wrong):
            assert np.abs(other - want).max() > 0.02 * np.abs(want).max(), f"wrong rule {i} would not show"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,softcap", [(4, 2, 16, 24, 4.0), (3, 3, 64, 64, 6.0), (4, 1, 128, 128, 3.0), (16, 2, 64, 64, 5.0)])
@pytest.mark.parametrize("cut", ["whole", "portions", "decode"])
def test_capped_attention_with_growing_queries_and_a_sink(dtype, H, G, dk, dv, softcap, cut):
    """The left one of two mixers: far keys stay in sight, the cap and the growth of the queries show."""
    from vllm_cpp_b200.config.registry import resolve_architecture
    from vllm_cpp_b200.parts.base import MIXERS, build_part
    width, n = 24, 190
    w, x = lone_keys(dtype, H, G, dk, dv, 16, (0, 15, 16, 77, 150), look_scale=1.0)
    m = cap(H, G, dk, dv, scale=1.0, softcap=softcap, q_temp=(0.9, 30))
    _, spec = resolve_architecture(config([par(m, ssd(2, 8, 4))], width=width))
    part = build_part(MIXERS, "mixer", spec.layers[0].mixer.params["left"], dtype=DT[dtype], device="cuda")
    part.load_params(part_weights(w, "", dtype, part))
    schedule = {"whole": [[("a", n)]], "portions": [[("a", t)] for t in (2, 30, 3, 64, 17, 2, 40, 32)],
                "decode": [[("a", 41)]] + [[("a", 1)] for _ in range(n - 41)]}[cut]
    got, _ = run_mixer(part, {"a": x}, schedule, page=16, pages=30, max_len=240, width_out=width)
    want = plain.capped_attention(x, w, "", m, 1e-5)
    assert np.abs(got["a"] - want).max() <= (3e-5 if dtype == "float32" else 2e-2) * np.abs(want).max()
    if cut == "whole":
        for other in (dict(m, softcap=None), dict(m, softcap=softcap * 1.5), dict(m, q_temp={"coef": 0.9, "every": 31}), dict(m, q_temp=None)):
            assert np.abs(plain.capped_attention(x, w, "", other, 1e-5) - want).max() > 0.01 * np.abs(want).max(), other


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", [att(6, 2, 12, 20, scale=0.5, bias_max=50, mask=(24, 5)), att(8, 2, 64, 64, scale=0.2, bias_max=60, mask=(33, 9)),
                                   att(4, 2, 128, 128, scale=0.12, bias_max=40, mask=(10, 17)), lat(3, 10, 6, 14, 20, 24), lat(2, 24, 2, 24, 33, 7, base=50.0),
                                   lat(4, 32, 16, 24, 48, 32, scale=0.2), lat(2, 40, 32, 48, 96, 56, scale=0.15, base=1e4), lat(4, 8, 12, 6, 12, 16, scaling=None),
                                   lat(4, 32, 64, 32, 192, 64, scale=0.12, base=1e4), lat(16, 32, 16, 32, 128, 64, scale=0.15, base=1e4),
                                   par(cap(4, 2, 16, 8), ssd(6, 8, 12, groups=3, norm_groups=2)), par(cap(4, 4, 64, 64), ssd(4, 16, 16, groups=2)),
                                   par(cap(3, 1, 10, 14), ssd(5, 7, 9, conv=1, norm_groups=5)), par(cap(2, 2, 64, 64), ssd(2, 64, 128, conv=3))])
def test_mixers_under_every_cut_with_slots_used_again(dtype, layer):
    width = 40
    w = rounded(plain.random_weights(config([layer], width=width), 4, sharp=1.5 if dtype == "float32" else 1.0), dtype)
    p = "l0.mix."
    part = part_of(layer, width, dtype)
    part.load_params(part_weights(w, p, dtype, part))
    rng = np.random.default_rng(6)
    x = {r: stored(rng.standard_normal((n, width)), dtype) for r, n in LENGTHS.items()}
    got, slots = run_mixer(part, x, SCHEDULE, page=8, pages=22, max_len=100)
    assert set(slots) == {0, 1}
    for r in x:
        want = plain.MIXERS[layer["type"]](x[r], w, p, layer["mixer"], 1e-5)
        assert np.abs(got[r] - want).max() <= (3e-5 if dtype == "float32" else 3e-2) * np.abs(want).max(), r


def test_the_stretched_rotation_and_the_sink_show():
    """Latent attention whose rotated parts alone decide, over a few hundred positions: what leaves out the stretching, the factor of
    cosine and sine, the rotation, or the sink is far from it."""
    width, n = 20, 300
    layer = lat(2, 4, 16, 8, 12, 10, scale=1.0, base=100.0, scaling=(6.0, 40, 4.0, 0.5))
    m = layer["mixer"]
    w = plain.random_weights(config([layer], width=width), 2)
    p = "l0.mix."
    w[p + "uk"] = w[p + "uk"] * 0.1
    part = part_of(layer, width, "float32")
    part.load_params(part_weights(w, p, "float32", part))
    x = np.random.default_rng(3).standard_normal((n, width))
    got, _ = run_mixer(part, {"a": stored(x, "float32")}, [[("a", 100)], [("a", 199)], [("a", 1)]], page=16, pages=30, max_len=400)
    want = plain.latent_attention(stored(x, "float32"), w, p, m, 1e-5)
    assert np.abs(got["a"] - want).max() <= 3e-5 * np.abs(want).max()
    s = m["rot"]["scaling"]
    for scaling in (None, dict(s, factor=5.0), dict(s, fast=2.0), dict(s, slow=0.25), dict(s, original=60)):
        other = dict(m, rot=dict(m["rot"], scaling=scaling))
        assert np.abs(plain.latent_attention(x, w, p, other, 1e-5) - want).max() > 0.02 * np.abs(want).max(), scaling
    no_sink = dict(w, **{p + "sink": np.full(2, -60.0)})
    assert np.abs(plain.latent_attention(x, no_sink, p, m, 1e-5) - want).max() > 0.02 * np.abs(want).max()


# ------------------------------------------------------------------ the state space in its dual form
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,N,P", [(4, 2, 32, 48), (2, 1, 128, 64), (3, 3, 16, 8), (6, 2, 64, 64), (2, 2, 72, 40), (5, 1, 9, 7), (1, 1, 200, 24), (2, 1, 512, 12),
                                     (4, 1, 128, 72), (150, 1, 24, 64), (2, 1, 3, 8), (3, 1, 8, 16), (1, 1, 1, 1)])
@pytest.mark.parametrize("walk", [True, False])
def test_state_dual_portions(dtype, H, G, N, P, walk):
    """Two requests side by side, portions at and around a chunk's edges, single tokens, slots that hold old numbers for others;
    the result beside the recurrence token by token, bfloat16 inputs included: the state and the sums are 32-bit."""
    from vllm_cpp_b200.csrc import ops
    if dtype == "float32" and not walk:
        pytest.skip("one kernel for float32")
    rng = np.random.default_rng(H * N + P)
    n = {"a": 210, "b": 131}
    x = {r: stored(rng.standard_normal((k, H * P)), dtype) for r, k in n.items()}
    B, C = ({r: stored(rng.standard_normal((k, G * N)), dtype) for r, k in n.items()} for _ in range(2))
    pre = {r: stored(-1.0 + rng.standard_normal((k, H)), dtype) for r, k in n.items()}
    bias, A, D = 0.3 * rng.standard_normal(H), -np.exp(rng.uniform(-3, 1.5, H)), rng.standard_normal(H)
    f = lambda a, dt=torch.float32: dev(np.asarray(a, dtype=np.float32), dt)
    state = torch.full((3, H, N, P), 7.0, device="cuda")
    slot = {"a": 2, "b": 0}
    for s in slot.values():
        state[s].zero_()
    got, at = {r: np.empty((k, H * P)) for r, k in n.items()}, {r: 0 for r in n}
    for step in ([("a", 64)], [("a", 65), ("b", 17)], [("a", 1), ("b", 1)], [("b", 63), ("a", 2)], [("a", 63)], [("b", 2)], [("a", 15), ("b", 48)]):
        lens = [k for _, k in step]
        take = lambda src, width: f(np.concatenate([src[r][at[r]: at[r] + k] for r, k in step]).reshape(-1, width), DT[dtype])
        y = torch.empty((sum(lens), H * P), device="cuda")
        # B and C beside x in one row, as the mixer has them
        row = torch.cat([take(x, H * P), take(B, G * N), take(C, G * N)], dim=1).contiguous()
        I, GN = H * P, G * N
        ops.state_dual(row[:, :I], row[:, I: I + GN], row[:, I + GN:], take(pre, H), f(bias), f(A * np.log2(np.e)), f(D), state, y,
                       dev(np.cumsum([0] + lens).astype(np.int32)), dev(np.array([slot[r] for r, _ in step], dtype=np.int32)), len(step), max(lens),
                       num_groups=G, walk=walk)
        out, t0 = y.cpu().numpy(), 0
        for r, k in step:
            got[r][at[r]: at[r] + k] = out[t0: t0 + k]
            at[r] += k
            t0 += k
    assert at == n and (state[1] == 7.0).all()
    for r, k in n.items():
        want, S = plain.decaying_outer_products(x[r].reshape(k, H, P), plain.softplus(pre[r] + bias), A, B[r].reshape(k, G, N), C[r].reshape(k, G, N), D)
        assert np.abs(got[r] - want.reshape(k, -1)).max() <= 2e-5 * np.abs(want).max(), r
        assert np.abs(state[slot[r]].cpu().numpy() - S).max() <= 2e-5 * np.abs(S).max(), r


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("steps", [[700], [7, 300, 1, 2, 390], [500] + [1] * 200, [64] * 10 + [60]])
def test_state_dual_remembers_a_token_of_hundreds_before(dtype, steps):
    """One loud token at the start, slow decays, silence after it: what is left of it after 700 tokens is what the equations say, and
    a head that forgets at once holds nothing (its decays underflow to zero without harm)."""
    from vllm_cpp_b200.csrc import ops
    H, N, P, n = 3, 32, 16, 700
    rng = np.random.default_rng(1)
    x, pre = np.zeros((n, H * P)), stored(-3.0 + 0.3 * rng.standard_normal((n, H)), dtype)
    x[0] = 40.0
    x[400] = 0.5
    B, C = stored(rng.standard_normal((n, N)), dtype), stored(rng.standard_normal((n, N)), dtype)
    A, D, bias = np.array([-0.02, -0.1, -3000.0]), rng.standard_normal(H), 0.1 * rng.standard_normal(H)
    f = lambda a, dt=torch.float32: dev(np.asarray(a, dtype=np.float32), dt)
    state, outs, at = torch.zeros((1, H, N, P), device="cuda"), [], 0
    for k in steps:
        s = slice(at, at + k)
        y = torch.empty((k, H * P), device="cuda")
        ops.state_dual(f(x[s], DT[dtype]), f(B[s], DT[dtype]), f(C[s], DT[dtype]), f(pre[s], DT[dtype]), f(bias), f(A * np.log2(np.e)), f(D), state, y,
                       dev(np.array([0, k], dtype=np.int32)), torch.zeros(1, dtype=torch.int32, device="cuda"), 1, k, num_groups=1)
        outs.append(y.cpu().numpy())
        at += k
    want, S = plain.decaying_outer_products(x.reshape(n, H, P), plain.softplus(pre + bias), A, B[:, None], C[:, None], D)
    got = np.concatenate(outs).reshape(n, H, P)
    assert np.isfinite(got).all() and np.abs(want[-1, 0]).max() > 1e-2
    assert np.abs(got - want).max() <= 2e-5 * np.abs(want).max()
    assert np.abs(got[-1, 0] - want[-1, 0]).max() <= 2e-4 * np.abs(want[-1, 0]).max()
    assert np.abs(got[5:395, 2]).max() <= 1e-6 and np.abs(state[0].cpu().numpy() - S).max() <= 1e-4 * np.abs(S).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("C,parts,n", [(48, 2, 5), (640, 5, 3), (512, 1, 4), (8192, 8, 2), (35, 5, 3), (8192, 1, 3), (2048, 16, 300)])
def test_gate_before_the_norm(dtype, C, parts, n):
    from vllm_cpp_b200.csrc import ops
    rng = np.random.default_rng(C)
    o, gate, w = rng.standard_normal((n, C)).astype(np.float32), stored(2 * rng.standard_normal((n, C)), dtype), (1 + 0.2 * rng.standard_normal(C)).astype(np.float32)
    out = torch.empty((n, C), dtype=DT[dtype], device="cuda")
    ops.gated_group_norm(dev(o), dev(gate, DT[dtype]), dev(w), out, group=C // parts, eps=1e-3, gate_act="silu", gate_first=True)
    norm = lambda v: plain.rms(v.reshape(n, parts, -1), 1e-3).reshape(n, C)
    want = norm(o * plain.silu(gate)) * w
    assert np.abs(out.float().cpu().numpy() - want).max() <= (2e-5 if dtype == "float32" else 5e-3) * np.abs(want).max()
    assert np.abs(norm(o) * plain.silu(gate) * w - want).max() > 0.1 * np.abs(want).max()


# ------------------------------------------------------------------ experts
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,mlp", [(64, moe(40, 8, 1, shared=24)), (72, moe(24, 5, 2)), (77, moe(13, 3, 3, shared=9)), (320, moe(96, 16, 4, shared=64))])
def test_experts_whose_weight_multiplies_what_they_read(dtype, width, mlp):
    from vllm_cpp_b200.csrc import ops
    from vllm_cpp_b200.parts.base import Workspace
    layer = att(2, 1, 8, 8, mlp=mlp)
    cfg = config([layer], width=width)
    w = rounded(plain.random_weights(cfg, 9), dtype)
    p = "l0.mlp."
    w[p + "router"] = w[p + "router"] * 3                            # scores well apart from 0.5 and from each other
    part = part_of(layer, width, dtype, slot="feed_forward")
    part.load_params(part_weights(w, p, dtype, part))
    for n in (1, 3, 40, 300):
        h = stored(np.random.default_rng(n).standard_normal((n, width)), dtype)
        s = -np.sort(-plain.sigmoid(h @ w[p + "router"].T), axis=-1)
        sure = np.ones(n, dtype=bool) if mlp["router"]["top"] == s.shape[1] else s[:, mlp["router"]["top"] - 1] - s[:, mlp["router"]["top"]] > 1e-5
        assert sure.mean() > 0.9
        out = torch.empty((n, width), dtype=DT[dtype], device="cuda")
        part.forward(dev(h, DT[dtype]), out, None, Workspace("cuda"))
        want = plain.routed_ff(h, w, p, mlp)
        got = out.float().cpu().numpy()
        assert np.abs(got - want)[sure].max() <= (3e-5 if dtype == "float32" else 2e-2) * np.abs(want).max(), n
    # where the weight goes matters
    ids, sc = plain.route(h, w[p + "router"], mlp["router"]["top"])
    after = np.stack([sum(a * plain.expert_ff(h[t:t + 1], w, f"{p}e{int(e)}.")[0] for e, a in zip(ids[t], sc[t])) for t in range(20)])
    before = np.stack([sum(plain.expert_ff(a * h[t:t + 1], w, f"{p}e{int(e)}.")[0] for e, a in zip(ids[t], sc[t])) for t in range(20)])
    assert np.abs(after - before).max() > 0.02 * np.abs(before).max()
    ops.check_status()


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_whole_prompts_and_the_first_tokens(tmp_path, name, dtype):
    cfg, w, _, cache, runner = build(tmp_path, name, dtype, 16)
    rp = Replayer(runner, cache)
    for n in (1, 2, 3, 47, 150):
        ids = ids_of(cfg, n, n)
        rp.step([(f"r{n}", ids, range(n))], end=[f"r{n}"])
        compare(rp.logits_of(f"r{n}", range(n)), plain.forward(cfg, w, ids), dtype, f"{name} whole {n}", slack_of(cfg, w, ids, dtype))
    assert cache.num_free_pages() == 16 and all(g.pool.num_free == g.pool.num_blocks for g in cache.paged)


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_the_stream_after_every_layer(tmp_path, name):
    cfg, w, _, cache, runner = build(tmp_path, name, "float32", 8)
    ids = ids_of(cfg, 60, 2)
    _, want = plain.forward(cfg, w, ids, return_layers=True)
    seen = []
    for blk in runner.model.blocks:
        def wrapped(residual, delta, *a, _inner=blk.forward, **k):
            result = _inner(residual, delta, *a, **k)
            seen.append((residual + delta if result is True else residual).float().cpu().numpy().copy())
            return result
        blk.forward = wrapped
    Replayer(runner, cache).step([("r", ids, [59])], end=["r"])
    assert len(seen) == want.shape[0]
    for i, (g, t) in enumerate(zip(seen, want)):
        assert np.abs(g - t).max() <= 3e-5 * np.abs(t).max(), f"layer {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_prefill_against_token_by_token_and_long_decoding(tmp_path, name, dtype):
    cfg, w, _, cache, runner = build(tmp_path, name, dtype, 24)
    n = 220
    ids = ids_of(cfg, n, 7)
    want, slack = plain.forward(cfg, w, ids), slack_of(cfg, w, ids, dtype)
    rp = Replayer(runner, cache)
    rp.step([("p", ids, range(n))], end=["p"])
    compare(rp.logits_of("p", range(n)), want, dtype, f"{name} prefill", slack)
    rp.step([("d", ids[:9], range(9))])
    for t in range(9, n):
        rp.step([("d", ids[t: t + 1], [0])])
    cache.free_request("d")
    compare(rp.logits_of("d", range(n)), want, dtype, f"{name} decode", slack)
    if dtype == "float32":
        a, b = rp.logits_of("p", range(n)), rp.logits_of("d", range(n))
        assert np.abs(a - b).max() <= 3e-5 * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_portions_down_to_two_tokens(tmp_path, name, dtype):
    cfg, w, _, cache, runner = build(tmp_path, name, dtype, 24)
    n = 150
    ids = ids_of(cfg, n, 9)
    want, slack = plain.forward(cfg, w, ids), slack_of(cfg, w, ids, dtype)
    for k, sizes in enumerate(([2] * 75, [5, 2, 31, 2, 17, 64, 3, 26], [16, 16, 1, 15, 33, 2, 67], [149, 1])):
        assert sum(sizes) == n
        rp, t = Replayer(runner, cache), 0
        for s in sizes:
            rp.step([(f"c{k}", ids[t: t + s], range(s))])
            t += s
        cache.free_request(f"c{k}")
        compare(rp.logits_of(f"c{k}", range(n)), want, dtype, f"{name} portions {sizes[:4]}", slack)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_unequal_requests_together_on_few_pages(tmp_path, name, dtype):
    """Up to three live requests of unequal length, portions beside single tokens, on so few pages and slots that both are used
    again by later requests; every request's logits are those it has alone."""
    cfg, w, _, cache, runner = build(tmp_path, name, dtype, 28, max_seqs=3)
    rng = np.random.default_rng(3)
    lengths = {"a": 90, "b": 3, "c": 140, "d": 33, "e": 64, "f": 1, "g": 120}
    ids = {r: ids_of(cfg, n, 60 + i) for i, (r, n) in enumerate(lengths.items())}
    want = {r: plain.forward(cfg, w, ids[r]) for r in ids}
    rp = Replayer(runner, cache)
    waiting, live, at = list(lengths), [], {}
    slots_seen = []
    while waiting or live:
        while waiting and len(live) < 3:
            live.append(waiting.pop(0))
            at[live[-1]] = 0
        entries, end = [], []
        for r in live:
            s = int(min(lengths[r] - at[r], 1 if at[r] > 40 else rng.choice([1, 2, 7, 16, 29])))
            entries.append((r, ids[r][at[r]: at[r] + s], range(s)))
            at[r] += s
            if at[r] == lengths[r]:
                end.append(r)
        rp.step(entries, end=[])
        slots_seen += [cache.slot(r) for r, _, _ in entries]
        for r in end:
            cache.free_request(r)
            compare(rp.logits_of(r, range(lengths[r])), want[r], dtype, f"{name} mixed {r}", slack_of(cfg, w, ids[r], dtype))
            live.remove(r)
    assert cache.num_free_pages() == 28 and len(set(slots_seen)) == 3
    assert all(g.pool.num_free == g.pool.num_blocks for g in cache.paged)


# larger layers: heads of 128 and 64 on the tensor-core kernels, windows of several key tiles, a state of 128 in several chunks
CFG_WIDE = config([att(8, 2, 128, 128, scale=0.088, bias_max=300, mask=(200, 20), mlp=dense(640)),
                   par(cap(8, 8, 64, 64, scale=0.125, softcap=15.0, q_temp=(0.3, 100)), ssd(16, 48, 128, groups=2, norm_groups=2), mlp=moe(128, 12, 2, shared=256)),
                   lat(6, 64, 32, 64, 96, 160, scale=0.1, base=1e4, scaling=(4.0, 256, 16.0, 1.0), mlp=moe(96, 4, 1, shared=128)),
                   att(6, 6, 64, 64, scale=0.125, bias_max=500, mask=(96, 65))], width=384, vocab=700)


def test_bfloat16_beside_float32_at_larger_sizes(tmp_path):
    """The same (bfloat16-valued) weights through the float32 engine, which the small configurations anchor to the plain
    implementation, and through the bfloat16 engine: a prompt of 650 tokens in two portions, then single tokens, beside a
    second request; captured decode steps too."""
    from vllm_cpp_b200 import EngineConfig
    from vllm_cpp_b200.engine import factory
    w = plain.round_to_bf16(plain.random_weights(CFG_WIDE, 3, sharp=1.0, decisive_routing=True))
    ids = {"a": ids_of(CFG_WIDE, 680, 5), "b": ids_of(CFG_WIDE, 70, 6)}
    steps = [[("a", 500)], [("a", 150), ("b", 40)]] + [[("a", 1), ("b", 1)]] * 30
    got = {}
    for dtype, graphs in (("float32", False), ("bfloat16", False), ("bfloat16", True)):
        folder = str(tmp_path / dtype)
        plain.write_model_folder(folder, CFG_WIDE, w, store="BF16" if dtype == "bfloat16" else "F32")
        ecfg = EngineConfig(model_path=folder, dtype=dtype, block_size=16, num_gpu_blocks=64, max_num_seqs=2, max_model_len=1024,
                            max_num_batched_tokens=512, use_cuda_graphs=graphs)
        _, cache, runner = factory.build(ecfg)
        rp, at = Replayer(runner, cache), {"a": 0, "b": 0}
        for step in steps:
            rp.step([(r, ids[r][at[r]: at[r] + n], range(n)) for r, n in step])
            for r, n in step:
                at[r] += n
        got[dtype, graphs] = {r: rp.logits_of(r, range(at[r])) for r in ids}
        del runner, cache
    for r in ids:
        for graphs in (False, True):
            compare(got["bfloat16", graphs][r], got["float32", False][r], "bfloat16", f"larger sizes {r}", plain.rounding_error(CFG_WIDE, w, ids[r], runs=1))


@pytest.mark.parametrize("dtype,name,pages", [("float32", "A", 24), ("bfloat16", "C", 24), ("float32", "B", 5), ("float32", "C", 24)])
def test_greedy_generation_through_the_entry_point(tmp_path, dtype, name, pages):
    """LLM.generate: the scheduler cuts the prompts under a small token budget, decode steps are captured and replayed; every
    generated token is the plain implementation's best, or within rounding of it.  On 5 pages requests are preempted and fed
    again from their first token: their state slots start from zero again."""
    from vllm_cpp_b200 import LLM, SamplingParams
    cfg, page = CONFIGS[name]
    weights = make_weights(cfg, 5, dtype)
    folder = str(tmp_path / f"gen_{dtype}")
    plain.write_model_folder(folder, cfg, weights, store="BF16" if dtype == "bfloat16" else "F32")
    llm = LLM(folder, dtype=dtype, block_size=page, num_gpu_blocks=pages, max_num_seqs=3, max_model_len=pages * page,
              max_num_batched_tokens=48)
    prompts = [ids_of(cfg, n, 500 + n) for n in (3, 41, 100, 17)]
    outs = llm.generate(prompts, SamplingParams(max_tokens=30, temperature=0.0, ignore_eos=True))
    if pages < 24:
        assert llm.engine.scheduler.num_preemptions > 0
    for p, o in zip(prompts, outs):
        assert len(o) == 30
        logits = plain.forward(cfg, weights, list(p) + list(o))
        for i, tok in enumerate(o):
            row = logits[len(p) - 1 + i]
            best = plain.greedy(row)
            assert tok == best or (row[best] - row[tok]) / np.abs(row).max() < (1e-3 if dtype == "float32" else 5e-2), (dtype, len(p), i)


def random_rufisun_config(rng):
    """Sizes with odd factors, all mixers and feed-forwards in any order, windows, kept tokens and chunks of every relation."""
    layers = []
    for _ in range(int(rng.integers(1, 6))):
        kind = rng.random()
        mlp = None if kind < 0.2 else dense(int(rng.integers(20, 160))) if kind < 0.5 else \
            moe(int(rng.integers(8, 60)), int(rng.integers(2, 9)), 1, None if rng.random() < 0.3 else int(rng.integers(8, 80)))
        if mlp is not None and mlp["kind"] == "moe":
            mlp["router"]["top"] = int(rng.integers(1, mlp["router"]["experts"] + 1))
        g, dk = int(rng.integers(1, 4)), int(rng.choice([8, 10, 16, 48, 64]))
        dv = dk if rng.random() < 0.4 else int(rng.choice([8, 14, 96]))
        heads = g * int(rng.integers(1, 4))
        which = rng.random()
        if which < 0.35:
            layers.append(att(heads, g, dk, dv, scale=float(rng.uniform(0.1, 0.4)), bias_max=float(rng.choice([25, 70.5, 300])),
                              mask=(int(rng.integers(1, 60)), int(rng.integers(0, 40))), mlp=mlp))
        elif which < 0.65:
            layers.append(lat(heads, dk, 2 * int(rng.integers(1, 10)), dv, int(rng.integers(8, 100)), int(rng.integers(6, 60)), scale=float(rng.uniform(0.1, 0.3)),
                              base=float(rng.choice([10.0, 500.0, 1e4, 1e6])),
                              scaling=None if rng.random() < 0.2 else (float(rng.uniform(1.5, 20)), int(rng.integers(20, 3000)), float(rng.uniform(2, 40)), float(rng.uniform(0.3, 2))),
                              mlp=mlp))
        else:
            groups, parts = int(rng.integers(1, 4)), int(rng.integers(1, 4))
            right = ssd(groups * parts * int(rng.integers(1, 3)), int(rng.choice([4, 8, 16, 20])), int(rng.choice([3, 8, 16, 40, 64])), groups,
                        conv=int(rng.integers(1, 6)), norm_groups=parts)
            layers.append(par(cap(heads, g, dk, dv, scale=float(rng.uniform(0.1, 0.4)), softcap=float(rng.uniform(2, 20)),
                                  q_temp=(float(rng.uniform(0, 1)), int(rng.integers(1, 50)))), right, (float(rng.uniform(0.3, 1.2)), float(rng.uniform(0.3, 1.2))), mlp=mlp))
    return config(layers, width=int(rng.choice([36, 50, 64, 90, 104, 136])), vocab=int(rng.integers(40, 500)), eps=float(rng.choice([1e-5, 1e-6, 1e-4])))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6])
def test_the_replay_program_on_configurations_drawn_at_random(tmp_path, seed, dtype):
    """bin/trace_run as a user calls it, on a configuration drawn at random, under a schedule drawn at random: JSON lines in,
    <step>.f32 files and 'done' lines out; a pool of as many tokens as live requests hold, four slots."""
    rng = np.random.default_rng(seed)
    cfg = random_rufisun_config(rng)
    weights = make_weights(cfg, seed, dtype)
    folder = str(tmp_path / "model")
    plain.write_model_folder(folder, cfg, weights, store="BF16" if dtype == "bfloat16" else "F32")
    lengths = {f"q{i}": int(n) for i, n in enumerate(rng.choice([1, 2, 30, 77, 150, 64], size=6))}
    ids = {r: ids_of(cfg, n, seed * 100 + i) for i, (r, n) in enumerate(lengths.items())}
    waiting, live, at, lines, asked = list(lengths), [], {}, [], []
    most = 0
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
            at[live[-1]] = 0
        most = max(most, sum(-(-lengths[r] // 64) * 64 for r in live))
        entries, end, rows = [], [], []
        for r in live:
            s = int(min(lengths[r] - at[r], 1 if at[r] > 50 else rng.choice([1, 2, 3, 16, 37, 64])))
            want = sorted(set(int(x) for x in rng.integers(0, s, size=min(s, 3))))
            entries.append({"id": r, "tokens": ids[r][at[r]: at[r] + s], "want": want})
            rows += [(r, at[r] + x) for x in want]
            at[r] += s
            if at[r] == lengths[r]:
                end.append(r)
        lines.append({"step": len(lines), "entries": entries, "end": end})
        asked.append(rows)
        live = [r for r in live if r not in end]
    out = tmp_path / "out"
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype,
                        "--out", str(out), "--max-tokens", str(most)],
                       input="".join(json.dumps(l) + "\n" for l in lines), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-3000:]
    assert [l for l in p.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(len(lines))]
    want = {r: plain.forward(cfg, weights, ids[r]) for r in ids}
    slack = {r: slack_of(cfg, weights, ids[r], dtype) for r in ids}
    got_rows, want_rows, slack_rows = [], [], []
    for i, rows in enumerate(asked):
        if rows:
            got = np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
            assert got.shape[0] == len(rows), f"step {i}: {got.shape[0]} rows written, {len(rows)} asked for"
            got_rows.append(got)
            want_rows.append(np.stack([want[r][t] for r, t in rows]))
            slack_rows += [0.0 if slack[r] is None else slack[r][t] for r, t in rows]
    compare(np.concatenate(got_rows), np.concatenate(want_rows), dtype, f"seed {seed}: {cfg['layers']}", slack_rows)


def test_command_line_and_sampling_options(tmp_path):
    """python -m vllm_cpp_b200.engine.cli on a Rufisun folder, the architecture taken from config.json or named by --arch: greedy
    ids are the plain implementation's; seeded sampling gives ids of the vocabulary, the same when asked again."""
    cfg, page = CONFIGS["B"]
    weights = make_weights(cfg, 8, "float32")
    folder = str(tmp_path / "cli_model")
    plain.write_model_folder(folder, cfg, weights, store="F32")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    prompt = ids_of(cfg, 21, 3)
    base = [sys.executable, "-m", "vllm_cpp_b200.engine.cli", "--model", folder, "--dtype", "float32", "--block-size", str(page),
            "--num-gpu-blocks", "24", "--max-num-seqs", "2", "--max-model-len", "128", "--max-num-batched-tokens", "64", "--ignore-eos",
            "--prompt-ids", ",".join(map(str, prompt))]
    env = dict(os.environ, PYTHONPATH=root)

    def run(extra):
        p = subprocess.run(base + extra, capture_output=True, text=True, timeout=600, env=env, cwd=root)
        assert p.returncode == 0, p.stderr[-3000:]
        return [int(t) for t in p.stdout.strip().splitlines()[-1].split(",")]

    greedy = run(["--max-tokens", "6", "--temperature", "0"])
    seq = list(prompt)
    for tok in greedy:
        logits = plain.forward(cfg, weights, seq)[-1]
        assert tok == plain.greedy(logits) or (logits.max() - logits[tok]) / np.abs(logits).max() < 1e-3
        seq.append(tok)
    options = ["--arch", "rufisun", "--max-tokens", "12", "--temperature", "0.9", "--top-k", "20", "--top-p", "0.9",
               "--repetition-penalty", "1.2", "--sample-seed", "5"]
    drawn = run(options)
    assert len(drawn) == 12 and all(0 <= t < cfg["vocab"] for t in drawn)
    assert run(options) == drawn
