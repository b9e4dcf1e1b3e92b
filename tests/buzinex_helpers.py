"""Tiny Buzinex configurations and model folders for the tests.

The configurations differ in every size and constant and avoid choices that would hide a mix-up: rotated, unrotated and value
sizes of a latent head differ, heads are one, several and no power of two, attentions have as many key/value heads as heads,
some, or one, key and value sizes differ, windows are one token, smaller than a page, larger than one and no multiple of one,
and several in one model, queries grow fast and slowly (and shrink), caps are low enough to matter, the decay's inner size is
smaller and larger than a head, layers of every kind come with and without a feed-forward, scales are away from one and
the logits' scale is below and above it.
"""
from __future__ import annotations

from pathlib import Path

import numpy as np
import torch

import plain_buzinex as plain


def latent(heads, dim, rot_dim, vdim, kv_rank, size, scale, base):
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                                "mask": {"size": size}, "rot": {"base": base, "dims": rot_dim}}


def full(heads, kv_heads, dim, vdim, scale, softcap, coef, every):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
                         "q_temp": {"coef": coef, "every": every}}


def wkv(heads, dim, rank):
    return "wkv", {"heads": heads, "dim": dim, "rank": rank}


def layer(mixer, ff=None):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(vocab, width, eps, scale, logit_scale, cap, layers):
    return {"architecture": "Buzinex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "logit_scale": logit_scale, "logit_softcap": cap, "layers": layers}


# sizes that are no multiples of 8
A = model(211, 36, 1e-5, 3.0, 0.6, 11.0, [
    layer(latent(3, 10, 6, 7, 20, 5, 0.31, 100.0), 28),
    layer(wkv(3, 6, 5), 20),
    layer(full(6, 3, 9, 11, 0.8, 7.0, 0.9, 3)),
    layer(latent(2, 4, 12, 5, 14, 19, 0.45, 3000.0)),
    layer(wkv(2, 11, 13)),
])
# one head, one window of a single token, one key/value head per head, queries that shrink
B = model(190, 64, 1e-6, 0.5, 2.5, 20.0, [
    layer(full(4, 4, 16, 24, 0.35, 9.0, -0.2, 20), 40),
    layer(latent(1, 16, 8, 24, 32, 1, 0.5, 50.0), 72),
    layer(wkv(1, 40, 24), 48),
    layer(latent(5, 8, 16, 16, 48, 33, 0.25, 20000.0)),
    layer(full(3, 1, 32, 32, 0.2, 6.0, 0.9, 64)),
])
# sizes that the tensor-core kernels of the bfloat16 path are built for, the projections of a recurrence in one launch
C = model(277, 128, 1e-5, 9.0, 0.8, 13.0, [
    layer(wkv(4, 64, 24), 96),
    layer(latent(8, 32, 16, 48, 64, 70, 0.15, 10000.0), 160),
    layer(full(8, 2, 64, 64, 0.125, 12.0, 0.35, 50)),
    layer(wkv(2, 64, 40)),
    layer(latent(4, 48, 32, 32, 96, 130, 0.12, 800.0), 104),
    layer(full(2, 2, 64, 128, 0.14, 30.0, 0.15, 7), 64),
])
CONFIGS = {"A": (A, 3, 16), "B": (B, 4, 8), "C": (C, 5, 16)}            # name -> (config.json, seed, page size)


def make_model_dir(base, name: str) -> Path:
    """A folder written by the package's random-weights mode, then made harder: matrices are scaled so that scores are well apart
    (a wrong key or a lost state must move the logits), decays run from fast to very slow (a state that is lost early
    shows hundreds of tokens later), bonuses, sinks, norms and blends are not small."""
    from sprout_lm_b200.config import parse_config
    from sprout_lm_b200.weights import write_random_model, write_safetensors
    from sprout_lm_b200.weights.safetensors_io import SafetensorsFile
    raw, seed, _ = CONFIGS[name]
    directory = write_random_model(Path(base) / f"buzinex_{name}", parse_config(raw), seed=seed)
    rng = np.random.default_rng(seed)
    uniform = lambda lo, hi, shape: torch.from_numpy(rng.uniform(lo, hi, tuple(shape)).astype(np.float32))
    spread = raw["width"] ** -0.5 / 0.02                          # a matrix scaled by this keeps a row's size
    tensors = {}
    handle = SafetensorsFile(directory / "model.safetensors")
    try:
        for key in handle.names():
            value = handle.tensor(key).float()
            if key.endswith(".w0"):
                value = torch.from_numpy(rng.permutation(np.linspace(-6.0, 0.5, value.numel())).astype(np.float32))
            elif key.endswith(".u"):
                value = uniform(-1.5, 2.0, value.shape)
            elif ".mu." in key:
                value = uniform(0.1, 0.9, value.shape)
            elif key.endswith(".sink"):
                value = uniform(-1.0, 2.5, value.shape)
            elif key.endswith((".q.norm", ".k.norm")):
                value = uniform(0.7, 2.2, value.shape)
            elif key.endswith("norm") or key.split(".")[-1].startswith("norm"):
                value = uniform(0.4, 1.6, value.shape)
            elif key == "embed":
                value = value * (1.5 / 0.02 * raw["width"] ** -0.5)
            elif key.endswith(".w2"):
                value = value * (1.2 / 0.02 * value.shape[1] ** -0.5)
            elif key.endswith((".uk", ".uv")):
                value = value * (1.8 / 0.02 * value.shape[1] ** -0.5)
            elif key.endswith((".mix.q", ".mix.dkv")):
                value = value * spread * 1.8
            elif value.dim() == 2:
                value = value * spread * 1.2
            tensors[key] = value.to(torch.bfloat16)
    finally:
        handle.close()
    write_safetensors(directory / "model.safetensors", tensors, metadata={"format": "pt"})
    return directory


_models: dict = {}
_logits: dict = {}


def plain_model(directory):
    """(config.json as a dict, name -> float64 array)."""
    key = str(directory)
    if key not in _models:
        _models[key] = plain.read_model_folder(str(directory))
    return _models[key]


def plain_logits(directory, tokens) -> np.ndarray:
    key = (str(directory), tuple(tokens))
    if key not in _logits:
        _logits[key] = plain.forward(*plain_model(directory), list(tokens))
    return _logits[key]


def rounding_moves(directory, tokens) -> np.ndarray:
    """Per position, how far the plain implementation's logits move (``relative``) at most when its matrix products read and
    write bfloat16, four times with a little noise before the rounding (where a head's output nearly cancels, its norm makes much
    of little, either way): what rounding alone does at that place of that model."""
    key = (str(directory), tuple(tokens), "rounded")
    if key not in _logits:
        want, moves = plain_logits(directory, tokens), []
        for seed in range(4):
            rng = np.random.default_rng(seed)
            with plain.rounding(lambda a: plain.to_bfloat16(a * (1.0 + (0.002 * rng.uniform(-1.0, 1.0, np.shape(a)) if seed else 0.0)))):
                moved = plain.forward(*plain_model(directory), list(tokens))
            moves.append([relative(a, b) for a, b in zip(moved, want)])
        _logits[key] = np.max(moves, axis=0)
    return _logits[key]


def plain_greedy(directory, prompt, new_tokens: int) -> list:
    history, out = list(prompt), []
    for _ in range(new_tokens):
        row = plain.forward(*plain_model(directory), history)[-1]
        out.append(int(np.argmax(row)))
        history.append(out[-1])
    return out


def relative(got, want) -> float:
    """Root mean square of got - want over the vocabulary, divided by that of want about its mean."""
    spread = float(np.sqrt(np.mean((want - want.mean()) ** 2)))
    return float(np.sqrt(np.mean((np.asarray(got, dtype=np.float64) - want) ** 2))) / max(spread, 1e-6)


def compare(directory, requests: dict, got: dict, tol: float, label: str, page: int, rounded: bool = False):
    """Every place that came back against the plain implementation, by ``relative``; a failure names the first wrong token
    and what is special about its place.  ``rounded`` (16-bit runs): a place's bar is ``tol`` or, where the model is touchy,
    three times what rounding the plain implementation's matrix products does there."""
    assert got, "no logits came back"
    worst = 0.0
    for rid, tokens in requests.items():
        want = plain_logits(directory, tokens)
        bars = np.maximum(tol, 3.0 * rounding_moves(directory, tokens)) if rounded else np.full(len(tokens), tol)
        for pos in range(len(tokens)):
            if (rid, pos) not in got:
                continue
            err = relative(got[(rid, pos)], want[pos])
            assert np.isfinite(err) and err <= bars[pos], \
                (f"{label}: request {rid} position {pos} of {len(tokens)} (position % {page} = {pos % page}) "
                 f"differs by {err:.3e} > {bars[pos]:.3e}")
            worst = max(worst, err)
    return worst
