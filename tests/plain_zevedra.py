"""A plain, slow Zevedra decoder in numpy float64: one function per mechanism, whole sequences at once, no cache.

It shares nothing with the package (its own safetensors reader included) and is what the framework's kernels, cache,
state slots and step function are compared with.  The model: a scaled token embedding plus a row of a table that the last
two tokens choose; layers with one-number norms before each sublayer and a multiplier on what a sublayer adds; two kinds of
mixer, each with softmax attention beside a recurrence (``parallel``: a window with rotated values beside the gated delta
rule; ``parallel_2``: every earlier position, a sink without a value, an elementwise gate, beside a recurrence whose forget
gate also decides what is written); routed experts whose weight multiplies their input; a span of layers that runs several
times with the same weights; a final norm and a head.
"""
from __future__ import annotations

import json
import math
import struct

import numpy as np


# ------------------------------------------------------------------------------------------------ files
def read_safetensors(path) -> dict:
    """name -> float64 array of a safetensors file: 8-byte length, JSON header, data."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        raw, shape = data[lo:hi], info["shape"]
        if info["dtype"] == "BF16":
            bits = np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16
            out[name] = bits.view(np.float32).astype(np.float64).reshape(shape)
        elif info["dtype"] == "F32":
            out[name] = np.frombuffer(raw, dtype="<f4").astype(np.float64).reshape(shape)
        else:
            raise ValueError(f"{name}: dtype {info['dtype']}")
    return out


def read_model_folder(folder):
    with open(f"{folder}/config.json") as f:
        config = json.load(f)
    return config, read_safetensors(f"{folder}/model.safetensors")


# ------------------------------------------------------------------------------------------------ small pieces
ROUND = None            # a function array -> array; set (see ``rounding``) to learn how far 16-bit matrix products move a result


def to_bfloat16(a):
    """Round to the nearest bfloat16 (ties to even), returned as float64."""
    bits = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    bits = (bits + 0x7FFF + ((bits >> 16) & 1)) & np.uint32(0xFFFF0000)
    return bits.view(np.float32).astype(np.float64)


class rounding:
    """``with rounding(to_bfloat16):`` every matrix product's input and output pass through the function."""

    def __init__(self, fn):
        self.fn = fn

    def __enter__(self):
        global ROUND
        self.before, ROUND = ROUND, self.fn

    def __exit__(self, *exc):
        global ROUND
        ROUND = self.before


def lin(x, weight, exact=False):
    """W x for every row of x (weights are stored [out, in]); ``exact``: never rounded (32-bit quantities)."""
    if ROUND is None or exact:
        return x @ weight.T
    return ROUND(ROUND(x) @ weight.T)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, dtype=np.float64)))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def unit_rms(x, eps):
    """x divided by its root mean square over the last axis (eps inside the root)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def short_conv(u, weight):
    """u [T, channels], weight [channels, taps]: y_t = sum_j weight[:, j] * u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], weight.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return sum(padded[j:j + T] * weight[:, j] for j in range(taps))


def rotate(x, positions, base, dims, interleaved):
    """x [T, heads, dim]: the first ``dims`` elements of each head turn by position * base^(-2i/dims); pair i is elements
    (2i, 2i + 1), or (i, i + dims / 2)."""
    if not dims:
        return x
    half = dims // 2
    angle = np.asarray(positions, dtype=np.float64)[:, None] * base ** (-2.0 * np.arange(half) / dims)
    cos, sin = np.cos(angle)[:, None, :], np.sin(angle)[:, None, :]
    first, second = (slice(0, dims, 2), slice(1, dims, 2)) if interleaved else (slice(0, half), slice(half, dims))
    out = x.copy()
    out[..., first] = x[..., first] * cos - x[..., second] * sin
    out[..., second] = x[..., second] * cos + x[..., first] * sin
    return out


def softmax_attention(q, k, v, scale, window=None, unit_sink=False):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V].  ``window``: position i sees j with 0 <= i - j < window;
    ``unit_sink``: one is added to every denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    seen = (back >= 0) & (back < (window or T))
    out = np.zeros((T, H, v.shape[2]))
    for head in range(H):
        g = head // (H // G)
        s = np.where(seen, (q[:, head] @ k[:, g].T) * scale, -np.inf)
        top = s.max(axis=1, keepdims=True)
        if unit_sink:
            top = np.maximum(top, 0.0)
        e = np.exp(s - top)
        total = e.sum(axis=1, keepdims=True) + (np.exp(-top) if unit_sink else 0.0)
        out[:, head] = (e / total) @ v[:, g]
    return out


# ------------------------------------------------------------------------------------------------ recurrences
def delta_rule(q, k, v, g, beta, state=None):
    """q, k [T, G, D], v [T, H, V], decays g and write strengths beta [T, H].  Per head, with the q and k of group
    h // (H / G): S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q.  Returns (o [T, H, V], S [H, D, V])."""
    T, H, V = v.shape
    G, D = k.shape[1:]
    S = np.zeros((H, D, V)) if state is None else state.copy()
    group = np.arange(H) // (H // G)
    out = np.zeros((T, H, V))
    for t in range(T):
        kt, qt = k[t, group], q[t, group]
        S = S * g[t][:, None, None]
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, kt))
        S = S + kt[:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, qt)
    return out, S


def forget_and_write(q, f, v, state=None):
    """q, f [T, H, D], v [T, H, V]: S <- diag(f) S + (1 - f) v^T, o = S^T q.  Returns (o [T, H, V], S [H, D, V])."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2])) if state is None else state.copy()
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out, S


# ------------------------------------------------------------------------------------------------ mixers
def window_attention(h, w, p, m, positions, eps):
    """Convolved projections, interleaved rotation, unit-length-like queries and keys, values that turn with their position
    and heads' outputs that turn back, a sliding window, a gate per head."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(lin(h, w[p + key]), w[p + key + ".conv"]) for key in ("q", "k", "v"))
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = unit_rms(rotate(q.reshape(T, H, D), positions, base, dims, True), eps)
    k = unit_rms(rotate(k.reshape(T, G, D), positions, base, dims, True), eps)
    v = rotate(v.reshape(T, G, V), positions, base, V, True)
    out = softmax_attention(q, k, v, m["scale"], window=m["mask"]["size"])
    out = rotate(out, -positions, base, V, True)
    out = out * sigmoid(lin(h, w[p + "g"]))[:, :, None]
    return lin(out.reshape(T, H * V), w[p + "o"])


def gated_delta(h, w, p, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(lin(h, w[p + key]), w[p + key + ".conv"])) for key in ("q", "k", "v"))

    def unit(x):
        return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)
    q, k = unit(q.reshape(T, G, D)) * D ** -0.5, unit(k.reshape(T, G, D))
    beta = sigmoid(lin(h, w[p + "b"], exact=True))
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(lin(h, w[p + "a"], exact=True) + w[p + "dt_bias"]))
    out, _ = delta_rule(q, k, v.reshape(T, H, V), g, beta)
    out = rms_norm(out, w[p + "norm"], eps) * silu(lin(h, w[p + "g"]).reshape(T, H, V))
    return lin(out.reshape(T, H * V), w[p + "o"])


def full_attention(h, w, p, m, positions, eps):
    """Query and key norms over the whole projection, half-split rotation, one added to the softmax's denominator, a gate
    per element."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(lin(h, w[p + "q"]), w[p + "q.norm"], eps).reshape(T, H, D)
    k = rms_norm(lin(h, w[p + "k"]), w[p + "k.norm"], eps).reshape(T, G, D)
    v = lin(h, w[p + "v"]).reshape(T, G, V)
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q, k = rotate(q, positions, base, dims, False), rotate(k, positions, base, dims, False)
    out = softmax_attention(q, k, v, m["scale"], unit_sink=True).reshape(T, H * V)
    return lin(out * sigmoid(lin(h, w[p + "g"])), w[p + "o"])


def hgrn2(h, w, p, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = silu(lin(h, w[p + "q"])).reshape(T, H, D)
    v = lin(h, w[p + "v"]).reshape(T, H, V)
    low = w[p + "lower"]
    f = low + (1.0 - low) * sigmoid(lin(h, w[p + "f"]) + w[p + "f.b"])
    out, _ = forget_and_write(q, f.reshape(T, H, D), v)
    return lin(rms_norm(out, w[p + "norm"], eps).reshape(T, H * V), w[p + "o"])


def mixer(h, w, p, kind, m, positions, eps):
    if kind == "parallel":
        return m["left_scale"] * window_attention(h, w, p + "left.", m["left"], positions, eps) \
            + m["right_scale"] * gated_delta(h, w, p + "right.", m["right"], eps)
    if kind == "parallel_2":
        left = rms_norm(full_attention(h, w, p + "left.", m["left"], positions, eps), w[p + "left.out"], eps)
        right = rms_norm(hgrn2(h, w, p + "right.", m["right"], eps), w[p + "right.out"], eps)
        return 0.5 * (left + right)
    raise ValueError(kind)


# ------------------------------------------------------------------------------------------------ feed-forward
def route(h, router, top):
    """(chosen experts [T, top], their scores [T, top]): sigmoid scores, the largest ones, not renormalized."""
    z = lin(h, router, exact=True)
    ids = np.argsort(-z, axis=1, kind="stable")[:, :top]
    return ids, sigmoid(np.take_along_axis(z, ids, axis=1))


def moe_mlp(h, w, p, mlp):
    """The weight multiplies the expert's input."""
    ids, scores = route(h, w[p + "router"], mlp["router"]["top"])
    out = np.zeros((h.shape[0], w[p + "e0.down"].shape[0]))
    for e in range(mlp["router"]["experts"]):
        rows, places = np.nonzero(ids == e)
        if len(rows) == 0:
            continue
        a = h[rows] * scores[rows, places][:, None]
        y = lin(silu(lin(a, w[f"{p}e{e}.gate"])) * lin(a, w[f"{p}e{e}.up"]), w[f"{p}e{e}.down"])
        np.add.at(out, rows, y)
    return out


# ------------------------------------------------------------------------------------------------ the model
def embed(config, w, tokens):
    spec = config["embedding"]
    x = w["embed"][tokens] * spec["scale"]
    bigram = spec.get("bigram")
    if bigram:
        before = np.concatenate([[0], tokens[:-1]])
        row = (before * bigram["mul_prev"] + tokens * bigram["mul_cur"]) % bigram["buckets"]
        row[0] = bigram["buckets"]
        x = x + w["bigram"][row]
    return x


def run_order(config):
    """(layer, pass number or None, first of its pass) for every layer run."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    order = [(i, None, False) for i in range(start)]
    for t in range(times):
        order += [(i, t, i == start) for i in range(start, stop)]
    return order + [(i, None, False) for i in range(stop, n)]


def layer_forward(x, config, w, index, positions):
    layer, eps, p, mult = config["layers"][index], config["norm"]["eps"], f"l{index}.", config["residual_mult"]
    x = x + mult * mixer(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["type"], layer["mixer"], positions, eps)
    if layer.get("mlp") is not None:
        x = x + mult * moe_mlp(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"])
    return x


def forward(config, w, tokens, return_layers=False):
    """Logits [tokens, vocab] of one sequence from position 0 (and the stream after every layer run)."""
    tokens = np.asarray(tokens, dtype=np.int64)
    positions = np.arange(len(tokens))
    first = x = embed(config, w, tokens)
    after = []
    for index, number, begins in run_order(config):
        if begins:
            if number > 0:
                x = x + first
            x = x + w["loop.step"][number]
        x = layer_forward(x, config, w, index, positions)
        after.append(x)
    logits = lin(rms_norm(x, w["final.norm"], config["norm"]["eps"]), w["head"])
    return (logits, np.stack(after)) if return_layers else logits
