"""A plain, slow implementation of the Kasuvik design in numpy (float64), one function per mechanism, written from
the design's equations.  It shares no code with the engine: the tests compare the engine with it.

The design.  A decoder whose residual stream starts as embedding * scale; every sublayer has an RMS norm before and one
after it, x += norm_b(sublayer(norm_a(x))), all gains plain.  Mixers:

  "general_delta"  a matrix of keys by values per head under a generalised delta rule: every token decays the matrix
                   per key channel, removes (at a rate per key channel) what the matrix held under the token's unit key, and
                   adds the outer product of the plain key and the value.  Each head's result is divided by its root mean
                   square; the concatenated heads get a gain and a sigmoid gate.
  "parallel"       two mixers on the same input.  Left: grouped-query softmax attention; q, k and v (with biases) pass a
                   short causal convolution, q and k a rotation of interleaved pairs, every head's scores have a factor of
                   their own, and a query sees a sliding window of tokens plus, for what lies before the window, one mean
                   key and value per block of ``pool`` tokens.  Right: a selective state space of one vector per channel.
                   The two results are normed over the model's width and averaged.

The feed-forward is a gated one with relu.
"""
import math

import numpy as np

from plain_gipinex import read_model_folder, read_safetensors, rms, rotate_pairs, round_to_bf16, sigmoid, write_model_folder  # noqa: F401

UNIT_EPS = 1e-6
DECAY_RATE = math.exp(-0.5)


# ------------------------------------------------------------- shapes and random weights
def kv_heads(m):
    return m.get("kv_heads") or m["heads"]


def tensor_shapes(cfg, rank=12):
    """name -> shape of every tensor a model of this configuration has; ``rank``: the inner width of the decay's products,
    which no configuration key gives."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,), "head": (cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        out[p + "norm1"] = out[p + "norm1b"] = (W,)
        q = p + "mix."
        if layer["type"] == "general_delta":
            C = m["heads"] * m["dim"]
            for t in ("r", "k", "v", "g", "a"):
                out[q + t] = (C, W)
            out.update({q + "a.b": (C,), q + "w1": (rank, W), q + "w2": (C, rank), q + "w0": (C,), q + "norm": (C,), q + "o": (W, C)})
        else:
            l, r = m["left"], m["right"]
            H, G = l["heads"], kv_heads(l)
            for t, c in (("q", H * l["dim"]), ("k", G * l["dim"]), ("v", G * l["vdim"])):
                out.update({f"{q}left.{t}": (c, W), f"{q}left.{t}.b": (c,), f"{q}left.{t}.conv": (c, l["conv"])})
            out.update({q + "left.temp": (H,), q + "left.o": (W, H * l["vdim"])})
            I, R, N = r["inner"], r["dt_rank"], r["state"]
            out.update({q + "right.in": (2 * I, W), q + "right.conv": (I, r["conv"]), q + "right.conv.b": (I,),
                        q + "right.x": (R + 2 * N, I), q + "right.dt": (I, R), q + "right.dt.b": (I,),
                        q + "right.A_log": (I, N), q + "right.D": (I,), q + "right.o": (W, I),
                        q + "left.out": (W,), q + "right.out": (W,)})
        mlp = layer.get("mlp")
        if mlp is not None:
            out.update({p + "norm2": (W,), p + "norm2b": (W,), p + "mlp.gate": (mlp["ff"], W), p + "mlp.up": (mlp["ff"], W),
                        p + "mlp.down": (W, mlp["ff"])})
    return out


def random_weights(cfg, seed, sharp=1.0, rank=12):
    """Matrices of standard deviation fan_in^(-1/2); queries and keys of the attention times ``sharp`` (peaked scores, so
    that a wrong key shows); decays and step sizes spread over their ranges."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        x = rng.standard_normal(shape)
        leaf = name.split(".", 1)[1] if name.startswith("l") and name[1].isdigit() else name
        last = leaf.split("mix.")[-1]
        if name == "embed":
            w = x
        elif name == "final.norm" or leaf.startswith("norm") or last in ("norm", "left.out", "right.out"):
            w = 1.0 + 0.1 * x
        elif last.endswith(".conv"):
            w = 0.4 * x
            w[:, -1] += 1.0
        elif last == "left.temp":
            w = 1.0 + 0.3 * x
        elif last == "right.A_log":
            w = np.log(np.linspace(0.5, 4.0, shape[1]))[None, :] + 0.2 * x
        elif last == "right.dt.b":
            w = -2.0 + x
        elif last == "right.D":
            w = 1.0 + 0.3 * x
        elif last in ("a.b", "w0"):
            w = x
        elif last.endswith(".b"):
            w = 0.2 * x
        else:
            w = x / math.sqrt(shape[1])
            if last in ("left.q", "left.k"):
                w = w * sharp
        out[name] = w
    return out


# ------------------------------------------------------------- mechanisms
_rounding = None        # inside ``rounded_like_bf16``: the generator of the perturbations


class rounded_like_bf16:
    """Inside this context every product's input and result carries a random relative error of up to half a bfloat16 unit: what
    any computation with bfloat16 activations may differ by.  Where a design divides by a root mean square that is nearly zero
    (a head whose first token has r . k near zero takes its sign from it), that is much more than elsewhere."""

    def __init__(self, seed):
        self.rng = np.random.default_rng(seed)

    def __enter__(self):
        global _rounding
        _rounding = self.rng

    def __exit__(self, *exc):
        global _rounding
        _rounding = None


def perturbed(x):
    return x if _rounding is None else x * (1.0 + _rounding.uniform(-1, 1, size=x.shape) * 2.0 ** -9)


def product(h, w):
    """W h for rows h."""
    return perturbed(perturbed(h) @ w.T)


def softplus(z):
    return np.where(z > 30, z, np.log1p(np.exp(np.minimum(z, 30))))


def silu(z):
    return z * sigmoid(z)


def normed(x, w, eps):
    return rms(x, eps) * w


def short_conv(x, taps, bias=None):
    """y[t] = sum_j taps[:, j] x[t - (J - 1) + j] (+ bias), zeros before the start.  x: [n, C]; taps: [C, J]."""
    n, J = x.shape[0], taps.shape[1]
    y = np.zeros_like(x)
    for t in range(n):
        for j in range(J):
            s = t - (J - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y if bias is None else y + bias


def pooled_visibility(i, size, pool):
    """(first visible token, number of visible blocks) of position i.  ``size`` None: every token; ``pool`` None: no blocks."""
    if size is None:
        return 0, 0
    first = max(0, i - size + 1)
    if not pool:
        return first, 0
    blocks = 0
    while (blocks + 1) * pool - 1 <= i - size:
        blocks += 1
    return first, blocks


def pooled_attention_core(q, k, v, scale, temp, size, pool):
    """q: [n, H, d]; k: [n, G, d]; v: [n, G, dv], as the cache holds them.  Returns [n, H, dv]."""
    n, H, _ = q.shape
    G = k.shape[1]
    nb = n // pool if pool else 0
    kb = np.stack([k[b * pool:(b + 1) * pool].mean(axis=0) for b in range(nb)]) if nb else k[:0]
    vb = np.stack([v[b * pool:(b + 1) * pool].mean(axis=0) for b in range(nb)]) if nb else v[:0]
    out = np.empty((n, H, v.shape[2]))
    for i in range(n):
        first, blocks = pooled_visibility(i, size, pool)
        for h in range(H):
            g = h // (H // G)
            keys = np.concatenate([kb[:blocks, g], k[first:i + 1, g]])
            vals = np.concatenate([vb[:blocks, g], v[first:i + 1, g]])
            s = keys @ q[i, h] * scale * temp[h]
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ vals
    return out


def windowed_attention(h, w, p, m, eps):
    """The left mixer of one request, whole."""
    n = h.shape[0]
    H, G, d, dv = m["heads"], kv_heads(m), m["dim"], m["vdim"]
    q, k, v = (perturbed(short_conv(product(h, w[p + t]) + w[p + t + ".b"], w[p + t + ".conv"])) for t in ("q", "k", "v"))
    q, k, v = q.reshape(n, H, d), k.reshape(n, G, d), v.reshape(n, G, dv)
    if m.get("rot"):
        pos = np.arange(n, dtype=np.float64)
        q, k = (rotate_pairs(x, pos, m["rot"]["base"], m["rot"]["dims"]) for x in (q, k))
    mask = m.get("mask") or {}
    o = pooled_attention_core(q, k, v, m["scale"], w[p + "temp"], mask.get("size"), mask.get("pool"))
    return product(o.reshape(n, H * dv), w[p + "o"])


def selective_scan_core(x, dt, A, B, C, D, S=None):
    """A token's step: every channel's row of S decays by e^(dt * its row of A), takes in (dt * x) B and is read by C; the token's
    own x joins times D.  Returns (y, S)."""
    S = np.zeros(A.shape) if S is None else S.copy()
    y = np.empty_like(x)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def selective_state(h, w, p, m, eps):
    """The right mixer of one request, whole."""
    I, R, N = m["inner"], m["dt_rank"], m["state"]
    xz = product(h, w[p + "in"])
    x, z = xz[:, :I], xz[:, I:]
    x = silu(short_conv(x, w[p + "conv"], w[p + "conv.b"]))
    low = product(x, w[p + "x"])
    dt = softplus(product(low[:, :R], w[p + "dt"]) + w[p + "dt.b"])
    y, _ = selective_scan_core(x, dt, -np.exp(w[p + "A_log"]), low[:, R:R + N], low[:, R + N:], w[p + "D"])
    return product(y * silu(z), w[p + "o"])


def parallel(h, w, p, m, eps):
    left = windowed_attention(h, w, p + "left.", m["left"], eps)
    right = selective_state(h, w, p + "right.", m["right"], eps)
    return 0.5 * (normed(left, w[p + "left.out"], eps) + normed(right, w[p + "right.out"], eps))


def general_delta_core(r, k, v, decay, removal, S=None):
    """r, k, decay, removal: [n, H, d]; v: [n, H, dv].  Returns (o [n, H, dv], S [H, d, dv])."""
    n, H, d = r.shape
    S = np.zeros((H, d, v.shape[2])) if S is None else S.copy()
    o = np.empty((n, H, v.shape[2]))
    for t in range(n):
        for h in range(H):
            u = k[t, h] / math.sqrt((k[t, h] ** 2).sum() + UNIT_EPS)
            held = u @ S[h]
            S[h] = decay[t, h][:, None] * S[h] - np.outer(removal[t, h] * u, held) + np.outer(k[t, h], v[t, h])
            o[t, h] = r[t, h] @ S[h]
    return o, S


def general_delta(h, w, p, m, eps):
    n, H, d = h.shape[0], m["heads"], m["dim"]
    r, k, v = (product(h, w[p + t]).reshape(n, H, d) for t in ("r", "k", "v"))
    decay = np.exp(-DECAY_RATE * sigmoid(product(np.tanh(product(h, w[p + "w1"])), w[p + "w2"]) + w[p + "w0"]))
    removal = sigmoid(product(h, w[p + "a"]) + w[p + "a.b"])
    o, _ = general_delta_core(r, k, v, decay.reshape(n, H, d), removal.reshape(n, H, d))
    o = rms(o, eps).reshape(n, H * d) * w[p + "norm"] * sigmoid(product(h, w[p + "g"]))
    return product(o, w[p + "o"])


def feed_forward(h, w, p):
    return product(np.maximum(product(h, w[p + "gate"]), 0.0) * product(h, w[p + "up"]), w[p + "down"])


MIXERS = {"general_delta": general_delta, "parallel": parallel}


def forward(cfg, w, ids, return_layers=False):
    """Logits [n, vocab] of one request's tokens, all at once."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(ids)] * cfg["embedding"]["scale"]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](normed(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
        x = x + normed(y, w[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            x = x + normed(feed_forward(normed(x, w[p + "norm2"], eps), w, p + "mlp."), w[p + "norm2b"], eps)
        after.append(x.copy())
    logits = product(normed(x, w["final.norm"], eps), w["head"])
    return (logits, np.stack(after)) if return_layers else logits


def rounding_error(cfg, w, ids, runs=4):
    """Per row of the logits, the largest error over all tokens that perturbations of bfloat16's size caused in ``runs`` tries."""
    want = forward(cfg, w, ids)
    worst = np.zeros(len(want))
    for seed in range(runs):
        with rounded_like_bf16(seed):
            worst = np.maximum(worst, np.abs(forward(cfg, w, ids) - want).max(axis=1))
    return worst


def greedy(logits):
    return int(np.argmax(logits))
