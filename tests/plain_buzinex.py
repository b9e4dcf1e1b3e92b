"""A plain, slow Buzinex decoder in numpy float64: one function per mechanism, whole sequences at once, no cache.

It shares nothing with the package (its own safetensors reader included) and is what the framework's kernels, cache,
state slots and step function are compared with.  The model: a scaled token embedding; layers with an RMS norm before and
after each sublayer; three kinds of mixer (latent attention over a sliding window with a sink; attention over every earlier
position with query and key norms, capped scores and queries that grow with their position; a recurrence with a decay per
channel and a bonus for the current token, whose inputs are blends with the token before); a silu-gated feed-forward, or
none; a final norm and the embedding table as the head, with a scale and a cap on the logits.
"""
from __future__ import annotations

import json
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


def lin(x, weight):
    """W x for every row of x (weights are stored [out, in])."""
    if ROUND is None:
        return x @ weight.T
    return ROUND(ROUND(x) @ weight.T)


def silu(z):
    z = np.asarray(z, dtype=np.float64)
    return z / (1.0 + np.exp(-z))


def unit_rms(x, eps):
    """x divided by its root mean square over the last axis (eps inside the root)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def soft_cap(x, cap):
    return cap * np.tanh(x / cap)


def rotate_pairs(x, positions, base):
    """x [T, heads, dims]: elements (2i, 2i + 1) turn by position * base^(-2i/dims)."""
    dims = x.shape[-1]
    if not dims:
        return x
    angle = np.asarray(positions, dtype=np.float64)[:, None] * base ** (-2.0 * np.arange(dims // 2) / dims)
    cos, sin = np.cos(angle)[:, None, :], np.sin(angle)[:, None, :]
    out = np.empty_like(x)
    out[..., 0::2] = x[..., 0::2] * cos - x[..., 1::2] * sin
    out[..., 1::2] = x[..., 1::2] * cos + x[..., 0::2] * sin
    return out


def softmax_rows(scores, sink=None):
    """Rows of scores (hidden places are -inf) to weights; ``sink``: exp(sink) joins the denominator."""
    top = scores.max(axis=1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(scores - top)
    return e / (e.sum(axis=1, keepdims=True) + (np.exp(sink - top) if sink is not None else 0.0))


def visible(T, window=None):
    """[T, T]: query i sees key j with 0 <= i - j (< window)."""
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (back >= 0) & (back < (window or T))


def latent_scores(q_plain, q_turned, k_plain, k_turned, scale):
    """One head's scores: q_plain [T, d] with k_plain [T, d], plus q_turned [T, r] with the key part k_turned [T, r]."""
    return (q_plain @ k_plain.T + q_turned @ k_turned.T) * scale


def query_growth(positions, coef, every):
    """What a query at position p is multiplied by: 1 + coef ln(floor((p + 1) / every) + 1)."""
    return 1.0 + coef * np.log(np.floor((np.asarray(positions, dtype=np.float64) + 1.0) / every) + 1.0)


# ------------------------------------------------------------------------------------------------ recurrence
def blend_with_before(h, share, before=None):
    """Row t: h_t + (h_(t-1) - h_t) * share; ``before`` is the row ahead of the first (zeros at the start)."""
    first = np.zeros((1, h.shape[1])) if before is None else before.reshape(1, -1)
    return h + (np.concatenate([first, h[:-1]]) - h) * share


def decay_with_bonus(r, k, v, w, u, state=None):
    """r, k, w [T, H, D], v [T, H, V], u [H, D].  Per head o_t = (S + diag(u) k_t v_t^T)^T r_t, then S <- diag(w_t) S + k_t v_t^T.
    Returns (o [T, H, V], S [H, D, V])."""
    T, H, D = r.shape
    S = np.zeros((H, D, v.shape[2])) if state is None else state.copy()
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        write = k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S + u[:, :, None] * write, r[t])
        S = w[t][:, :, None] * S + write
    return out, S


# ------------------------------------------------------------------------------------------------ mixers
def latent_attention(h, w, p, m, positions, eps):
    T = h.shape[0]
    H, D, R, V, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = lin(h, w[p + "q"]).reshape(T, H, D + R)
    down = lin(h, w[p + "dkv"])
    c = rms_norm(down[:, :rank], w[p + "dkv.norm"], eps)
    base = m["rot"]["base"]
    k_turned = rotate_pairs(down[:, None, rank:], positions, base)[:, 0]
    q_turned = rotate_pairs(q[..., D:], positions, base)
    k_plain = lin(c, w[p + "uk"]).reshape(T, H, D)
    v = lin(c, w[p + "uv"]).reshape(T, H, V)
    seen = visible(T, m["mask"]["size"])
    out = np.zeros((T, H, V))
    for head in range(H):
        s = latent_scores(q[:, head, :D], q_turned[:, head], k_plain[:, head], k_turned, m["scale"])
        out[:, head] = softmax_rows(np.where(seen, s, -np.inf), w[p + "sink"][head]) @ v[:, head]
    return lin(out.reshape(T, H * V), w[p + "o"])


def attention(h, w, p, m, positions, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(lin(h, w[p + "q"]).reshape(T, H, D), w[p + "q.norm"], eps)
    k = rms_norm(lin(h, w[p + "k"]).reshape(T, G, D), w[p + "k.norm"], eps)
    v = lin(h, w[p + "v"]).reshape(T, G, V)
    q = q * query_growth(positions, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    seen = visible(T)
    out = np.zeros((T, H, V))
    for head in range(H):
        g = head // (H // G)
        s = soft_cap((q[:, head] @ k[:, g].T) * m["scale"], m["softcap"])
        out[:, head] = softmax_rows(np.where(seen, s, -np.inf)) @ v[:, g]
    return lin(out.reshape(T, H * V), w[p + "o"])


def wkv(h, w, p, m, eps):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    mixed = {key: blend_with_before(h, w[p + "mu." + key]) for key in ("r", "k", "v", "g", "w")}
    r, k, v = (lin(mixed[key], w[p + key]).reshape(T, H, D) for key in ("r", "k", "v"))
    gate = silu(lin(mixed["g"], w[p + "g"]))
    decay = np.exp(-np.exp(lin(np.tanh(lin(mixed["w"], w[p + "w1"])), w[p + "w2"]) + w[p + "w0"])).reshape(T, H, D)
    out, _ = decay_with_bonus(r, k, v, decay, w[p + "u"])
    return lin(unit_rms(out, eps).reshape(T, H * D) * w[p + "norm"] * gate, w[p + "o"])


def mixer(h, w, p, kind, m, positions, eps):
    if kind == "latent_attention":
        return latent_attention(h, w, p, m, positions, eps)
    if kind == "attention":
        return attention(h, w, p, m, positions, eps)
    if kind == "wkv":
        return wkv(h, w, p, m, eps)
    raise ValueError(kind)


def gated_mlp(h, w, p):
    return lin(silu(lin(h, w[p + "gate"])) * lin(h, w[p + "up"]), w[p + "down"])


# ------------------------------------------------------------------------------------------------ the model
def layer_forward(x, config, w, index, positions):
    layer, eps, p = config["layers"][index], config["norm"]["eps"], f"l{index}."
    y = mixer(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["type"], layer["mixer"], positions, eps)
    x = x + rms_norm(y, w[p + "norm1b"], eps)
    if layer.get("mlp") is not None:
        x = x + rms_norm(gated_mlp(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp."), w[p + "norm2b"], eps)
    return x


def head(config, w, x):
    logits = lin(rms_norm(x, w["final.norm"], config["norm"]["eps"]), w["embed"]) * config["logit_scale"]
    return soft_cap(logits, config["logit_softcap"])


def forward(config, w, tokens, return_layers=False):
    """Logits [tokens, vocab] of one sequence from position 0 (and the stream after every layer)."""
    tokens = np.asarray(tokens, dtype=np.int64)
    positions = np.arange(len(tokens))
    x = w["embed"][tokens] * config["embedding"]["scale"]
    after = []
    for index in range(len(config["layers"])):
        x = layer_forward(x, config, w, index, positions)
        after.append(x)
    logits = head(config, w, x)
    return (logits, np.stack(after)) if return_layers else logits
