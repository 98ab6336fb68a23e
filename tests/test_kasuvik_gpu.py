"""The Kasuvik design on the GPU against the plain implementation of plain_kasuvik.py: each mechanism alone (convolution +
rotation + cache write, the means of blocks, attention at the edges of its window and of its blocks, the selective state
space, the generalised delta rule, the joined norms, relu in the feed-forward), then whole models under every way of cutting
the work and greedy generation through the engine's entry point, the replay program and the command line.  Configurations
and weights are made here."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_kasuvik as plain
from helpers import MEAN_TOL, TOL, Replayer, kv_pos
from test_kasuvik_config import att, config, gdelta, par, sel
from test_lutodra_gpu import DT, LENGTHS, SCHEDULE, dev, mixer_harness, run_mixer, stored

pytestmark = pytest.mark.gpu

# every branch: head and value sizes that differ, groups of query heads, windows and blocks of several sizes (a block longer
# than the window, blocks of one token), no blocks, no mask, no rotation, convolutions of 1 to 9 taps, layers without feed-forward
CFG_A = config([par(att(6, 2, 12, 20, conv=3, scale=0.35, rot=(8, 300.0), mask=(24, 5)), sel(40, 6, 7), ff=96),
                gdelta(3, 16, ff=64),
                par(att(4, 1, 16, 8, conv=4, scale=0.25, rot=(16, 5000.0), mask=(9, 14)), sel(72, 16, 5, conv=2))], width=64, vocab=200, scale=0.6)
CFG_B = config([gdelta(5, 8), par(att(3, 3, 10, 14, conv=1, scale=0.4, rot=None, mask=(17, 1)), sel(33, 3, 4, conv=5), ff=50),
                par(att(2, 2, 24, 24, conv=2, scale=0.2, rot=(24, 50.0), mask=(40, 0)), sel(20, 33, 2, conv=1), ff=72),
                par(att(5, 1, 8, 12, conv=9, scale=0.3, rot=(2, 20.0), mask=None), sel(24, 8, 3, conv=10))], width=72, vocab=301, eps=1e-6, scale=1.3)
CFG_C = config([par(att(8, 2, 64, 64, conv=3, scale=0.125, rot=(32, 1e4), mask=(37, 6)), sel(48, 16, 6), ff=80), gdelta(1, 40, ff=56),
                par(att(4, 4, 128, 128, conv=3, scale=0.09, rot=(128, 1e5), mask=(70, 11)), sel(64, 4, 3), ff=40)], width=88, vocab=264)
CONFIGS = {"A": (CFG_A, 16), "B": (CFG_B, 32), "C": (CFG_C, 16)}
SHARP = {"float32": 2.0, "bfloat16": 1.0}


def compare(got, want, dtype, what="", slack=None):
    """Rows of logits against the plain implementation's: every row within TOL of the largest logit, in bfloat16 plus twice what
    perturbations of bfloat16's size cause in the plain implementation at that row (``slack``, plain.rounding_error: a head's
    and a mixer's result are normed by themselves, and where their terms nearly cancel, the norm multiplies the rounding); the
    mean error within MEAN_TOL over the rows, with the same addition."""
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
    return None if dtype == "float32" else plain.rounding_error(cfg, w, ids, runs=4 if len(ids) > 8 else 24)


def make_weights(cfg, seed, dtype):
    w = plain.random_weights(cfg, seed, sharp=SHARP[dtype])
    return plain.round_to_bf16(w) if dtype == "bfloat16" else w


def ids_of(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()


def build(tmp_path, name, dtype, num_pages, seed=1, max_seqs=4, graphs=False, cfg_page=None):
    from vllm_cpp_b200 import EngineConfig
    from vllm_cpp_b200.engine import factory
    cfg, page = cfg_page or CONFIGS[name]
    weights = make_weights(cfg, seed, dtype)
    folder = str(tmp_path / f"kasuvik_{name}_{dtype}")
    plain.write_model_folder(folder, cfg, weights, store="BF16" if dtype == "bfloat16" else "F32")
    ecfg = EngineConfig(model_path=folder, dtype=dtype, block_size=page, num_gpu_blocks=num_pages, max_num_seqs=max_seqs,
                        max_model_len=num_pages * page, max_num_batched_tokens=1024, use_cuda_graphs=graphs)
    model, cache, runner = factory.build(ecfg)
    return cfg, weights, folder, cache, runner


def part_weights(w, p, dtype, part):
    """The tensors of ``part`` out of plain weights under prefix p, in the types the loader gives them."""
    return {n: dev(np.asarray(w[p + n], dtype=np.float32), torch.float32 if ps.role != "matrix" else DT[dtype])
            for n, ps in part.param_specs().items()}


def mixer_weights(cfg, seed, dtype, sharp=1.0):
    w = plain.random_weights(cfg, seed, sharp=sharp)
    return plain.round_to_bf16(w) if dtype == "bfloat16" else w


def attention_part(m, dtype, width):
    from vllm_cpp_b200.config.model_spec import PartSpec
    from vllm_cpp_b200.parts import model  # noqa: F401  (registers the parts)
    from vllm_cpp_b200.parts.pooled_attention import PooledWindowAttention
    rot, mask = m.get("rot"), m.get("mask") or {}
    position = PartSpec("none") if not rot else PartSpec("scaled_rope", {"theta": rot["base"], "rotary_dim": rot["dims"], "pairing": "interleaved",
                                                                         "scaling": None})
    return PooledWindowAttention(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], m["scale"], mask.get("size", 0),
                                 mask.get("pool", 0), position, DT[dtype], "cuda")


# ------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,J,rot,page", [(6, 2, 12, 20, 3, 8, 16), (4, 1, 16, 8, 4, 16, 8), (3, 3, 7, 5, 2, 4, 16), (2, 2, 24, 24, 1, 0, 16),
                                                  (2, 1, 64, 64, 5, 64, 16), (3, 1, 8, 12, 11, 2, 24)])
def test_convolution_rotation_and_cache_write_under_every_cut(dtype, H, G, dk, dv, J, rot, page):
    """Queries out and keys and values in the pages, request by request, whatever the portions; slots are used again by later
    requests; the projection's bias is not added to the zeros before the start."""
    from vllm_cpp_b200.csrc import ops
    from vllm_cpp_b200.cache.manager import CacheManager
    from vllm_cpp_b200.parts.base import PagedKVSpec
    rng = np.random.default_rng(H * dk + J)
    C, row = H * dk + G * (dk + dv), max(dk, dv)
    taps, bias = rng.standard_normal((C, J)).astype(np.float32), rng.standard_normal(C).astype(np.float32)
    temp = (1 + 0.5 * rng.standard_normal(H)).astype(np.float32)
    base = 200.0
    inv = dev((base ** (-2.0 * np.arange(rot // 2) / max(rot, 1))).astype(np.float32)) if rot else None
    x = {r: stored(rng.standard_normal((n, C)), dtype) for r, n in LENGTHS.items()}
    want = {}
    for r, a in x.items():
        y = plain.short_conv(a + bias, taps.astype(np.float64))
        q, k, v = y[:, :H * dk].reshape(-1, H, dk), y[:, H * dk:(H + G) * dk].reshape(-1, G, dk), y[:, (H + G) * dk:].reshape(-1, G, dv)
        if rot:
            q, k = (plain.rotate_pairs(u, np.arange(len(a), dtype=np.float64), base, rot) for u in (q, k))
        want[r] = (q * temp[None, :, None], k, v)
    cm = CacheManager([PagedKVSpec(G, row)], page, 14, 2, DT[dtype], "cuda")
    pages = cm.views()[0].pages.view(14, -1)
    state = torch.zeros((2, max(1, J - 1), C), device="cuda")
    at = {r: 0 for r in x}
    esize = pages.element_size()
    tol = 3e-5 if dtype == "float32" else 1e-2
    for entries in SCHEDULE:
        for r, _ in entries:
            if r not in cm.requests:
                cm.add_request(r)
                state[cm.slot(r)].zero_()
        for r, n in entries:
            cm.reserve(r, n)
        i32 = lambda a: dev(np.asarray(a, dtype=np.int32))
        proj = dev(np.concatenate([x[r][at[r]: at[r] + n] for r, n in entries]), DT[dtype])
        q = torch.empty((proj.shape[0], H * dk), dtype=DT[dtype], device="cuda")
        table = cm.table_rows(0, 14)[[cm.slot(r) for r, _ in entries]]
        ops.conv_rope_cache_write(proj, dev(bias), dev(taps), state, inv, dev(temp), q, pages, i32(np.cumsum([0] + [n for _, n in entries])),
                                  i32(np.concatenate([np.arange(at[r], at[r] + n) for r, n in entries])), i32([cm.slot(r) for r, _ in entries]),
                                  i32(table), len(entries), max(n for _, n in entries), num_heads=H, num_kv_heads=G, head_dim=dk, v_head_dim=dv,
                                  row=row, page_size=page)
        ops.check_status()
        got, t0 = q.float().cpu().numpy().reshape(-1, H, dk), 0
        held = pages.float().cpu().numpy().reshape(14, 2, G, page * row)
        for r, n in entries:
            wq, wk, wv = want[r]
            sl = slice(at[r], at[r] + n)
            assert np.abs(got[t0:t0 + n] - wq[sl]).max() <= tol * max(1.0, np.abs(wq).max()), (r, at[r])
            for t in range(at[r], at[r] + n):
                pg, slot = cm.table(r, 0)[t // page], t % page
                where = kv_pos(row, esize, slot, page)
                for g in range(G):
                    assert np.abs(held[pg, 0, g][where][:dk] - wk[t, g]).max() <= tol * max(1.0, np.abs(wk).max())
                    assert np.abs(held[pg, 1, g][where][:dv] - wv[t, g]).max() <= tol * max(1.0, np.abs(wv).max())
            t0 += n
            at[r] += n
            cm.commit(r, n)
            if at[r] == LENGTHS[r]:
                cm.free_request(r)
    # the taps' order and the bias matter here
    flipped = plain.short_conv(x["a"] + bias, taps[:, ::-1].astype(np.float64))
    if J > 1:
        assert np.abs(flipped - plain.short_conv(x["a"] + bias, taps.astype(np.float64))).max() > 0.1


# a lone key that every query looks for: its weight jumps where it enters or leaves what a query sees
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,size,pool,page", [(4, 2, 16, 24, 20, 6, 8), (2, 1, 8, 8, 5, 13, 16), (3, 3, 12, 4, 1, 1, 16), (8, 2, 64, 64, 37, 6, 16),
                                                      (4, 1, 128, 128, 64, 16, 16), (4, 4, 64, 64, 130, 7, 8), (2, 2, 16, 16, 24, 0, 8),
                                                      (16, 1, 64, 64, 9, 3, 32), (6, 2, 128, 128, 3, 1, 16)])
@pytest.mark.parametrize("cut", ["whole", "portions", "decode"])
def test_attention_just_inside_and_just_outside_its_window_and_blocks(dtype, H, G, dk, dv, size, pool, page, cut):
    """Through the mixer: tokens whose keys stand out, at page, window and block borders.  The engine agrees with the plain
    rule at every position, and every wrong rule (a window one token longer or shorter, blocks one token early or late, a
    block size one off, no blocks) is far from it at some position."""
    width, n, m, w, x, q, k, v = lone_keys(dtype, H, G, dk, dv, size, pool, page)
    part = attention_part(m, dtype, width)
    part.load_params(part_weights(w, "", dtype, part))
    schedule = {"whole": [[("a", n)]], "portions": [[("a", t)] for t in (2, 30, 3, 64, 17, 2, 40, 32)],
                "decode": [[("a", 41)]] + [[("a", 1)] for _ in range(n - 41)]}[cut]
    got, _ = run_mixer(part, {"a": x}, schedule, page=page, pages=30, max_len=240, width_out=width)
    core = lambda s, p: plain.pooled_attention_core(q, k, v, 1.0, w["temp"], s, p).reshape(n, -1) @ w["o"].T
    want = core(size, pool)
    assert np.abs(got["a"] - want).max() <= (3e-5 if dtype == "float32" else 2e-2) * np.abs(want).max()
    if cut == "whole":
        for i, other in enumerate(wrong_rules(core, size, pool)):
            assert np.abs(other - want).max() > 0.04 * np.abs(want).max(), f"wrong rule {i} would not show"


def lone_keys(dtype, H, G, dk, dv, size, pool, page):
    width, n = 24, 190
    rng = np.random.default_rng(size * 10 + pool)
    m = att(H, G, dk, dv, conv=1, scale=1.0, rot=None, mask=(size, pool))
    look = rng.standard_normal(dk)
    look /= np.linalg.norm(look)
    w = {"q": np.zeros((H * dk, width)), "k": np.zeros((G * dk, width)), "v": rng.standard_normal((G * dv, width)) / np.sqrt(width),
         "o": rng.standard_normal((width, H * dv)) / np.sqrt(H * dv), "temp": np.linspace(0.8, 1.2, H),
         "q.b": np.tile(look * 3.0, H), "k.b": np.zeros(G * dk), "v.b": 0.1 * rng.standard_normal(G * dv)}
    w["k"][:, 0] = np.tile(look * 2.0, G)
    for t, c in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
        w[t + ".conv"] = np.ones((c, 1))
    if dtype == "bfloat16":
        w = plain.round_to_bf16(w)
    x = rng.standard_normal((n, width))
    x[:, 0] = 0.0
    for mark in (page - 1, 2 * max(pool, 1) + page) if size > 60 else (page - 1, 2 * max(pool, 1) + page, n // 2):
        x[mark, 0] = 1.0 + 0.8 * max(pool, 1)               # in a block's mean it is divided by the block's size
    x = stored(x, dtype)
    q, k, v = ((x @ w[t].T + w[t + ".b"]).reshape(n, -1, d) for t, d in (("q", dk), ("k", dk), ("v", dv)))
    return width, n, m, w, x, q, k, v


def wrong_rules(core, size, pool):
    """What rules that are one off give.  (Blocks of one token are the tokens themselves: where the window ends does not show.)"""
    out = []
    if pool != 1:
        out += [core(size + 1, pool)] + ([core(size - 1, pool)] if size > 1 else [])
    if pool:
        out += [core(size, 0), core(size, pool + 1)] + ([core(size, pool - 1)] if pool > 1 else [])
    if pool > 1:
        real = plain.pooled_visibility
        for shift in (-1, 1):                        # a block that is seen one token late, or one token early
            plain.pooled_visibility = lambda i, s, p, d=shift: (real(i, s, p)[0], real(max(0, i + d), s, p)[1])
            try:
                out.append(core(size, pool))
            finally:
                plain.pooled_visibility = real
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", [att(6, 2, 12, 20, conv=3, scale=0.5, rot=(8, 300.0), mask=(24, 5)), att(8, 2, 64, 64, conv=4, scale=0.2, rot=(32, 1e4), mask=(33, 9)),
                               att(4, 2, 128, 128, conv=2, scale=0.12, rot=(128, 1e5), mask=(70, 12)), att(4, 4, 64, 64, conv=3, scale=0.2, mask=(11, 0)),
                               att(2, 1, 10, 6, conv=2, scale=0.5, mask=None)])
def test_attention_mixer_under_every_cut_with_slots_used_again(dtype, m):
    width = 40
    w = plain.random_weights(config([par(m, sel(8, 2, 2))], width=width), 4, sharp=1.5)
    w = plain.round_to_bf16(w) if dtype == "bfloat16" else w
    p = "l0.mix.left."
    part = attention_part(m, dtype, width)
    part.load_params(part_weights(w, p, dtype, part))
    rng = np.random.default_rng(6)
    x = {r: stored(rng.standard_normal((n, width)), dtype) for r, n in LENGTHS.items()}
    got, slots = run_mixer(part, x, SCHEDULE, page=8, pages=22, max_len=100)
    assert set(slots) == {0, 1}
    for r in x:
        want = plain.windowed_attention(x[r], w, p, m, 1e-5)
        assert np.abs(got[r] - want).max() <= (3e-5 if dtype == "float32" else 3e-2) * np.abs(want).max(), r


def test_block_means_lie_in_their_rows_and_pages():
    """The rows of the blocks' pages are the means of the cached keys and values, each made once, by the step that brings the
    block's last token."""
    from vllm_cpp_b200.csrc import ops
    from vllm_cpp_b200.engine.runner import StepEntry
    from vllm_cpp_b200.parts.base import Workspace
    m, width, page = att(2, 2, 8, 8, conv=1, scale=0.3, rot=None, mask=(3, 5)), 16, 4
    w = plain.random_weights(config([par(m, sel(8, 2, 2))], width=width), 2)
    part = attention_part(m, "float32", width)
    part.load_params(part_weights(w, "l0.mix.left.", "float32", part))
    cache, runner = mixer_harness(part, page, 20, 80)
    pages = runner.views[0].views[1].pages
    cache.add_request("a")
    rng = np.random.default_rng(0)
    x, ws, at = rng.standard_normal((70, width)), Workspace("cuda"), 0
    k = ((x @ w["l0.mix.left.k"].T + w["l0.mix.left.k.b"]) * w["l0.mix.left.k.conv"][:, 0]).reshape(70, 2, 8)
    for n in (3, 1, 1, 4, 22, 1, 9, 29):
        step = runner._prepare([StepEntry("a", [0] * n, [])])
        out = torch.empty((n, width), device="cuda")
        part.forward(dev(x[at: at + n], torch.float32), out, step, runner.views[0], True, ws)
        cache.commit("a", n)
        ws.reset()
        at += n
        held = pages.cpu().numpy().reshape(pages.shape[0], 2, 2, -1)
        table = cache.table("a", 1)
        assert len(table) == -(-(at // 5) // page)
        for b in range(at // 5):
            for g in range(2):
                row = held[table[b // page], 0, g][kv_pos(8, 4, b % page, page)]
                assert np.abs(row - k[5 * b: 5 * b + 5, g].mean(axis=0)).max() < 1e-5
    ops.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("inner,N,rank,conv", [(40, 16, 5, 4), (33, 5, 7, 2), (130, 32, 3, 1), (20, 3, 2, 9), (24, 64, 4, 3), (17, 130, 3, 3), (64, 1, 1, 4),
                                               (16, 300, 2, 2), (48, 8, 6, 4)])
def test_selective_state_under_every_cut_with_slots_used_again(dtype, inner, N, rank, conv):
    from vllm_cpp_b200.parts.selective_state import SelectiveStateSpace
    width = 32
    w = mixer_weights(config([par(att(2, 1, 8, 8), sel(inner, N, rank, conv))], width=width), inner + N, dtype)
    p = "l0.mix.right."
    part = SelectiveStateSpace(width, inner, N, rank, conv, DT[dtype], "cuda")
    part.load_params(part_weights(w, p, dtype, part))
    rng = np.random.default_rng(N)
    x = {r: stored(rng.standard_normal((n, width)), dtype) for r, n in LENGTHS.items()}
    got, slots = run_mixer(part, x, SCHEDULE)
    assert set(slots) == {0, 1}
    m = {"inner": inner, "state": N, "dt_rank": rank, "conv": conv}
    for r in x:
        want = plain.selective_state(x[r], w, p, m, 1e-5)
        assert np.abs(got[r] - want).max() <= (3e-5 if dtype == "float32" else 3e-2) * np.abs(want).max(), r


@pytest.mark.parametrize("steps", [[600], [7, 300, 1, 2, 290], [500] + [1] * 100])
def test_selective_state_remembers_a_token_of_hundreds_before(steps):
    """One loud token at the start, slow decays, silence after it: what is left of it after 600 tokens is what the equations say
    (a state that is lost, or decays once too often, is far off), and the gate and the direct term are there."""
    from vllm_cpp_b200.csrc import ops
    I, N, n = 12, 6, 600
    rng = np.random.default_rng(1)
    x, dt_pre = np.zeros((n, I)), -5.0 + 0.3 * rng.standard_normal((n, I))
    x[0] = 40.0
    x[400] = 0.5
    B, C, z = rng.standard_normal((n, N)), rng.standard_normal((n, N)), 1.0 + rng.random((n, I))
    A, D, bias = -(0.05 + 0.2 * rng.random((I, N))), rng.standard_normal(I), 0.1 * rng.standard_normal(I)
    f = lambda a: dev(np.asarray(a, dtype=np.float32))
    state, out = torch.zeros((1, I, N), device="cuda"), torch.empty((n, I), device="cuda")
    at = 0
    slot = torch.zeros(1, dtype=torch.int32, device="cuda")
    for k in steps:
        s = slice(at, at + k)
        o = torch.empty((k, I), device="cuda")
        ops.selective_scan(f(x[s]), f(dt_pre[s]), f(B[s]), f(C[s]), f(z[s]), f(bias), f(A * np.log2(np.e)), f(D), state, o,
                           dev(np.array([0, k], dtype=np.int32)), slot, 1, k)
        out[s] = o
        at += k
    y, S = plain.selective_scan_core(x, plain.softplus(dt_pre + bias), A, B, C, D)
    want = y * plain.silu(z)
    assert np.abs(want[-1]).max() > 1e-2
    assert np.abs(out.cpu().numpy() - want).max() <= 2e-5 * np.abs(want).max()
    assert np.abs(out.cpu().numpy()[-1] - want[-1]).max() <= 1e-4 * np.abs(want[-1]).max()
    assert np.abs(state[0].cpu().numpy() - S).max() <= 1e-4 * np.abs(S).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,dk,dv,rank", [(3, 16, 16, 12), (1, 40, 8, 5), (4, 8, 33, 16), (2, 64, 64, 8), (1, 128, 40, 3), (2, 20, 20, 1), (1, 300, 12, 4),
                                          (5, 4, 4, 7)])
def test_general_delta_under_every_cut_with_slots_used_again(dtype, H, dk, dv, rank):
    from vllm_cpp_b200.parts.general_delta import GeneralDeltaRule
    width = 36
    rng = np.random.default_rng(H * dk)
    p = ""
    kk, vv = H * dk, H * dv
    shapes = {"r": (kk, width), "k": (kk, width), "v": (vv, width), "g": (vv, width), "a": (kk, width), "w1": (rank, width), "w2": (kk, rank), "o": (width, vv)}
    w = {t: rng.standard_normal(s) / np.sqrt(s[1]) for t, s in shapes.items()}
    w.update({"a.b": rng.standard_normal(kk), "w0": rng.standard_normal(kk), "norm": 1 + 0.2 * rng.standard_normal(vv)})
    w = plain.round_to_bf16(w) if dtype == "bfloat16" else w
    part = GeneralDeltaRule(width, H, dk, dv, plain.DECAY_RATE, 1e-5, DT[dtype], "cuda")
    part.load_params(part_weights(w, p, dtype, part))
    assert part.rank == rank
    x = {r: stored(rng.standard_normal((n, width)), dtype) for r, n in LENGTHS.items()}
    got, slots = run_mixer(part, x, SCHEDULE)
    assert set(slots) == {0, 1}
    for r, h in x.items():
        n = len(h)
        rr, k, a, z = ((h @ w[t].T).reshape(n, H, dk) for t in ("r", "k", "a", "a"))
        decay = np.exp(-plain.DECAY_RATE * plain.sigmoid(np.tanh(h @ w["w1"].T) @ w["w2"].T + w["w0"])).reshape(n, H, dk)
        removal = plain.sigmoid(h @ w["a"].T + w["a.b"]).reshape(n, H, dk)
        o, _ = plain.general_delta_core(rr, k, (h @ w["v"].T).reshape(n, H, dv), decay, removal)
        want = (plain.rms(o, 1e-5).reshape(n, vv) * w["norm"] * plain.sigmoid(h @ w["g"].T)) @ w["o"].T
        # a head's result is normed by itself: small heads whose terms nearly cancel multiply the rounding
        err = np.abs(got[r] - want).max(axis=1) / np.abs(want).max()
        tol = 5e-5 if dtype == "float32" else 4e-2
        assert np.quantile(err, 0.9) <= tol and err.max() <= 4 * tol, (r, err.max())


@pytest.mark.parametrize("steps", [[400], [7, 200, 1, 2, 190], [300] + [1] * 100, [2] * 200])
def test_general_delta_finds_a_key_written_hundreds_of_tokens_before(steps):
    """A key written early and asked for at the end: no decay on its channels, no removal by the keys between, then one token
    that removes it (so that rate, unit key and the order of read and write all show), float32."""
    from vllm_cpp_b200.csrc import ops
    H, dk, dv, n, rate = 2, 24, 10, 400, 3.0
    rng = np.random.default_rng(3)
    r, k, v = rng.standard_normal((n, H, dk)), rng.standard_normal((n, H, dk)), rng.standard_normal((n, H, dv))
    k[:, :, :8] = 0.0                                   # channels of their own for the far key
    k[5, :, :8] = 2.0 * rng.standard_normal((H, 8))
    k[5, :, 8:] = 0.0
    k[395] = 0.7 * k[5]                                 # removes and rewrites what was held
    z = np.full((n, H, dk), 0.5)
    z[:, :, :8] = -40.0                                 # exp(-rate * sigmoid(-40)) is 1: they never decay
    a_pre = rng.standard_normal((n, H, dk))
    r[390] = r[399] = 0.0
    r[390, :, :8] = r[399, :, :8] = k[5, :, :8]
    f = lambda a: dev(np.asarray(a, dtype=np.float32).reshape(a.shape[0], -1))
    state, at = torch.zeros((1, H, dk, dv), device="cuda"), 0
    outs = []
    for s in steps:
        sl = slice(at, at + s)
        o = torch.empty((s, H * dv), device="cuda")
        work = torch.empty(ops.general_delta_work(s, H, dk, dv), device="cuda")
        ops.general_delta(f(r[sl]), f(k[sl]), f(v[sl]), f(a_pre[sl]), f(z[sl]), None, None, state, o, dev(np.array([0, s], dtype=np.int32)),
                          torch.zeros(1, dtype=torch.int32, device="cuda"), 1, s, num_heads=H, rate=rate, unit_eps=plain.UNIT_EPS, work=work)
        outs.append(o.cpu().numpy())
        at += s
    got = np.concatenate(outs).reshape(n, H, dv)
    decay, removal = np.exp(-rate * plain.sigmoid(z)), plain.sigmoid(a_pre)
    want, S = plain.general_delta_core(r, k, v, decay, removal)
    held = (k[5, :, :8] ** 2).sum(axis=-1)[:, None] * v[5]
    assert np.abs(want[390] - held).max() < 1e-3 and np.abs(want[399] - held).max() > 1.0      # there, and then replaced
    assert np.abs(got - want).max() <= 2e-5 * np.abs(want).max()
    assert np.abs(got[390] - want[390]).max() <= 1e-4 * np.abs(want[390]).max()
    assert np.abs(state[0].cpu().numpy() - S).max() <= 1e-4 * np.abs(S).max()
    # rules that look alike are far from it
    for wrong in (lambda: plain.general_delta_core(r, k, v, decay, np.ones_like(removal)), lambda: plain.general_delta_core(r, k / 2, v, decay, removal)):
        assert np.abs(wrong()[0] - want).max() > 0.05 * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,n", [(72, 5), (77, 3), (320, 7), (2504, 2), (4096, 3), (9000, 2)])
def test_two_results_normed_joined_and_added(dtype, width, n):
    from vllm_cpp_b200.csrc import ops
    rng = np.random.default_rng(width)
    a, b = stored(3 * rng.standard_normal((n, width)), dtype), stored(0.05 * rng.standard_normal((n, width)), dtype)
    b[0] *= 1e-3                                                        # eps decides here
    b = stored(b, dtype)
    gains = [(1 + 0.3 * rng.standard_normal(width)).astype(np.float32) for _ in range(4)]
    x = rng.standard_normal((n, width)).astype(np.float32)
    y = 0.5 * plain.normed(a, gains[0], 1e-5) + 0.25 * plain.normed(b, gains[1], 1e-5)
    ga = [dev(g) for g in gains]
    da, db = dev(a, DT[dtype]), dev(b, DT[dtype])
    tol = 1e-5 if dtype == "float32" else 1e-2
    out = torch.empty_like(da)
    ops.pair_norm(da, db, ga[0], ga[1], 0.5, 0.25, 1e-5, out)
    assert np.abs(out.float().cpu().numpy() - y).max() <= tol * np.abs(y).max()
    new = x + plain.normed(y, gains[2], 1e-6)
    for with_next in (True, False):
        dx = dev(x)
        ops.pair_norm(da, db, ga[0], ga[1], 0.5, 0.25, 1e-5, out if with_next else None, x=dx, gain=ga[2], eps=1e-6,
                      next_gain=ga[3] if with_next else None, next_eps=1e-4)
        assert np.abs(dx.cpu().numpy() - new).max() <= 1e-5 * np.abs(new).max()            # float in both precisions
        if with_next:
            nxt = plain.normed(new, gains[3], 1e-4)
            assert np.abs(out.float().cpu().numpy() - nxt).max() <= tol * np.abs(nxt).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,ff", [(64, 96), (72, 50), (320, 384)])
@pytest.mark.parametrize("fused", [True, False])
def test_relu_feed_forward(dtype, width, ff, fused):
    """Few and many tokens; the product with relu in its epilogue (bfloat16, few tokens) and the kernel after the product."""
    from vllm_cpp_b200.csrc import ops
    from vllm_cpp_b200.parts.base import Workspace
    from vllm_cpp_b200.parts.mlp import GatedMLP
    if fused and (dtype == "float32" or width % 8):
        pytest.skip("the fused form is bfloat16")
    rng = np.random.default_rng(width)
    w = {"gate": rng.standard_normal((ff, width)) / np.sqrt(width), "up": rng.standard_normal((ff, width)) / np.sqrt(width),
         "down": rng.standard_normal((width, ff)) / np.sqrt(ff)}
    w = plain.round_to_bf16(w) if dtype == "bfloat16" else w
    part = GatedMLP(width, ff, "relu", DT[dtype], "cuda", tensor_names=("gate", "up", "down"))
    part.load_params({k: dev(v.astype(np.float32), DT[dtype]) for k, v in w.items()})
    if fused:
        ops.tile_weights(part.w_gate_up, ff)
        ops.forget_choices(2 * ff, width)
    for n in (1, 9, 40, 100, 200):
        h = stored(rng.standard_normal((n, width)), dtype)
        assert not fused or ops.linear_gated_fuses(n, part.w_gate_up) == (n <= 128)
        out = torch.empty((n, width), dtype=DT[dtype], device="cuda")
        part.forward(dev(h, DT[dtype]), out, None, Workspace("cuda"))
        want = plain.feed_forward(h, w, "")
        assert np.abs(out.float().cpu().numpy() - want).max() <= (2e-5 if dtype == "float32" else 2e-2) * np.abs(want).max(), n
    ops.check_status()
    if fused:
        ops.drop_tiled_weights(part.w_gate_up)


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


def test_the_stream_after_every_layer(tmp_path):
    cfg, w, _, cache, runner = build(tmp_path, "A", "float32", 8)
    ids = ids_of(cfg, 60, 2)
    _, want = plain.forward(cfg, w, ids, return_layers=True)
    seen = []
    for blk in runner.model.blocks:
        def wrapped(residual, *a, _inner=blk.forward, **k):
            result = _inner(residual, *a, **k)
            seen.append(residual.float().cpu().numpy().copy())
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


# larger layers: heads of 128 and 64 on the tensor-core kernels, windows of several key tiles, a state of 16, delta heads of 64
CFG_WIDE = config([par(att(8, 2, 128, 128, conv=4, scale=0.088, rot=(128, 1e5), mask=(200, 16)), sel(512, 16, 24), ff=640),
                   gdelta(6, 64, ff=512),
                   par(att(6, 6, 64, 64, conv=3, scale=0.125, rot=(32, 1e4), mask=(96, 7)), sel(320, 64, 12), ff=None),
                   gdelta(2, 128, ff=256)], width=384, vocab=700)


def test_bfloat16_beside_float32_at_larger_sizes(tmp_path):
    """The same (bfloat16-valued) weights through the float32 engine, which the small configurations anchor to the plain
    implementation, and through the bfloat16 engine: a prompt of 650 tokens in two portions, then single tokens, beside a
    second request; captured decode steps too."""
    from vllm_cpp_b200 import EngineConfig
    from vllm_cpp_b200.engine import factory
    w = plain.round_to_bf16(plain.random_weights(CFG_WIDE, 3, sharp=1.0))
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
            compare(got["bfloat16", graphs][r], got["float32", False][r], "bfloat16", f"larger sizes {r}", slack_of(CFG_WIDE, w, ids[r], "bfloat16"))


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


def random_kasuvik_config(rng):
    """Sizes with odd factors, both mixers in any order, windows and blocks of every relation, with and without rotation, mask,
    blocks and feed-forward.  (Delta heads have eight channels and more: a head's result is normed by itself.)"""
    layers = []
    for _ in range(int(rng.integers(1, 5))):
        ff = None if rng.random() < 0.25 else int(rng.integers(20, 160))
        if rng.random() < 0.4:
            layers.append(gdelta(int(rng.integers(1, 6)), int(rng.choice([8, 12, 16, 24, 33, 64])), ff=ff))
            continue
        g, dk = int(rng.integers(1, 4)), int(rng.choice([8, 10, 16, 48, 64]))
        dims = int(rng.choice([0, 2, dk // 2 // 2 * 2, dk]))
        mask = None if rng.random() < 0.15 else (int(rng.integers(1, 60)), 0 if rng.random() < 0.2 else int(rng.integers(1, 20)))
        layers.append(par(att(g * int(rng.integers(1, 4)), g, dk, dk if rng.random() < 0.4 else int(rng.choice([8, 14, 96])), conv=int(rng.integers(1, 6)),
                              scale=float(rng.uniform(0.1, 0.4)), rot=(dims, float(rng.choice([10.0, 500.0, 1e4, 1e6]))) if dims else None, mask=mask),
                          sel(int(rng.integers(8, 90)), int(rng.choice([1, 4, 7, 16, 32, 40])), int(rng.integers(1, 12)), conv=int(rng.integers(1, 6))), ff=ff))
    return config(layers, width=int(rng.choice([36, 50, 64, 90, 104, 136])), vocab=int(rng.integers(40, 500)), scale=float(rng.uniform(0.3, 2)),
                  eps=float(rng.choice([1e-5, 1e-6, 1e-4])))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6])
def test_the_replay_program_on_configurations_drawn_at_random(tmp_path, seed, dtype):
    """bin/trace_run as a user calls it, on a configuration drawn at random, under a schedule drawn at random: JSON lines in,
    <step>.f32 files and 'done' lines out; a pool of as many tokens as live requests hold, four slots."""
    rng = np.random.default_rng(seed)
    cfg = random_kasuvik_config(rng)
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
    """python -m vllm_cpp_b200.engine.cli on a Kasuvik folder, the architecture taken from config.json or named by --arch: greedy
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
    options = ["--arch", "kasuvik", "--max-tokens", "12", "--temperature", "0.9", "--top-k", "20", "--top-p", "0.9",
               "--repetition-penalty", "1.2", "--sample-seed", "5"]
    drawn = run(options)
    assert len(drawn) == 12 and all(0 <= t < cfg["vocab"] for t in drawn)
    assert run(options) == drawn
