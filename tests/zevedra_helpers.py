"""Tiny Zevedra configurations and model folders for the tests.

The configurations differ in every size and constant and avoid choices that would hide a mix-up: key and value sizes of a head
differ, attentions have as many key/value heads as heads, half as many, or one, recurrences share a query and key among
several heads or do not, convolutions have one to six taps and differ between the two mixers of a layer, the rotated width
is the whole vector, a part of it, or nothing, windows are smaller than a page, larger than one, and no multiple of one,
scales and multipliers are away from one and differ (one is negative), tokens take one expert or several, a layer has no
feed-forward, the loop covers the first layers, inner layers or nothing and runs two or three times, and one model has no
table of token pairs.
"""
from __future__ import annotations

from pathlib import Path

import numpy as np
import torch

import plain_zevedra as plain


def window(heads, kv_heads, dim, vdim, conv, size, scale, rot):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": size}, "scale": scale,
            "rot": {"base": rot[0], "dims": rot[1]}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def parallel(left, right, left_scale, right_scale):
    return "parallel", {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def parallel_2(heads, kv_heads, dim, vdim, scale, rot, right):
    return "parallel_2", {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                   "rot": {"base": rot[0], "dims": rot[1]}},
                          "right": {"heads": right[0], "dim": right[1], "vdim": right[2]}}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(mixer, mlp):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


# sizes that are no multiples of 8; inner layers run three times
A = {"architecture": "Zevedra", "vocab": 203, "width": 36, "norm": {"eps": 1e-5}, "residual_mult": 0.9,
     "embedding": {"scale": 3.0, "bigram": {"buckets": 97, "mul_prev": 11, "mul_cur": 5}},
     "loop": {"start": 1, "stop": 3, "times": 3},
     "layers": [
         layer(parallel(window(4, 2, 6, 10, 3, 5, 1.7, (100.0, 4)), delta(3, 1, 7, 5, 2), 0.7, 1.1), moe(5, 2, 12)),
         layer(parallel_2(3, 3, 8, 6, 0.6, (50.0, 8), (2, 5, 9)), None),
         layer(parallel(window(2, 1, 12, 4, 2, 9, 1.1, (700.0, 12)), delta(2, 2, 4, 11, 4), 1.2, -0.6), moe(4, 1, 20)),
         layer(parallel_2(2, 1, 10, 12, 0.4, (3000.0, 6), (3, 12, 4)), moe(7, 3, 9)),
     ]}
# no loop and no table of pairs; single taps, no rotation of the keys, a multiplier above one
B = {"architecture": "Zevedra", "vocab": 190, "width": 64, "norm": {"eps": 1e-6}, "residual_mult": 1.3, "embedding": {"scale": 0.5},
     "layers": [
         layer(parallel_2(4, 2, 16, 24, 0.35, (3000.0, 10), (2, 16, 16)), moe(6, 1, 24)),
         layer(parallel(window(4, 4, 16, 16, 6, 33, 0.25, (20000.0, 0)), delta(4, 2, 16, 24, 1), 0.5, 0.9), moe(4, 3, 16)),
         layer(parallel(window(6, 2, 8, 20, 1, 70, 0.4, (60.0, 8)), delta(1, 1, 20, 16, 5), 1.0, 0.7), None),
     ]}
# sizes that the tensor-core kernels of the bfloat16 path are built for; the first two layers run twice
C = {"architecture": "Zevedra", "vocab": 277, "width": 128, "norm": {"eps": 1e-5}, "residual_mult": 0.6,
     "embedding": {"scale": 9.0, "bigram": {"buckets": 400, "mul_prev": 40009, "mul_cur": 101}},
     "loop": {"start": 0, "stop": 2, "times": 2},
     "layers": [
         layer(parallel(window(8, 2, 64, 128, 4, 100, 0.11, (10000.0, 32)), delta(4, 1, 48, 64, 3), 0.8, 0.5), moe(8, 2, 32)),
         layer(parallel_2(2, 2, 96, 96, 0.12, (30000.0, 64), (2, 64, 40)), moe(4, 2, 40)),
         layer(parallel(window(4, 1, 32, 64, 2, 70, 0.2, (2000.0, 32)), delta(2, 2, 64, 32, 4), 0.6, 0.9), moe(6, 1, 64)),
     ]}
CONFIGS = {"A": (A, 3, 16), "B": (B, 4, 8), "C": (C, 5, 16)}            # name -> (config.json, seed, page size)
MIXER_SCALE = {"A": 8.0, "B": 6.0, "C": 4.0}
EXPERT_SCALE = {"A": 6.0, "B": 4.5, "C": 3.0}            # small enough that a nearly tied choice of experts is no landslide


def make_model_dir(base, name: str) -> Path:
    """A folder written by the package's random-weights mode, then made harder: matrices are scaled up so that every part is
    a large share of the stream (a wrong key or a lost state must move the logits), decays run from fast to very slow (a
    state that is lost early shows hundreds of tokens later), norms, taps, passes' vectors and pair rows are not small, and the
    routers' scores are well apart."""
    from sprout_lm_b200.config import parse_config
    from sprout_lm_b200.weights import write_random_model, write_safetensors
    from sprout_lm_b200.weights.safetensors_io import SafetensorsFile
    raw, seed, _ = CONFIGS[name]
    directory = write_random_model(Path(base) / f"zevedra_{name}", parse_config(raw), seed=seed)
    rng = np.random.default_rng(seed)
    uniform = lambda lo, hi, n: torch.from_numpy(rng.uniform(lo, hi, n).astype(np.float32))
    tensors = {}
    handle = SafetensorsFile(directory / "model.safetensors")
    try:
        for key in handle.names():
            value = handle.tensor(key).float()
            n = value.numel()
            if key.endswith(".A_log"):
                value = torch.from_numpy(rng.permutation(np.linspace(-4.0, 0.5, n)).astype(np.float32))
            elif key.endswith(".dt_bias"):
                value = uniform(-2.0, 1.0, n)
            elif key.endswith(".f.b"):
                value = torch.from_numpy(rng.permutation(np.linspace(-1.0, 6.0, n)).astype(np.float32))
            elif key.endswith(".lower"):
                value = uniform(0.0, 0.9, n)
            elif key.endswith((".q.norm", ".k.norm", ".mix.right.norm", ".left.out", ".right.out")):
                value = uniform(0.4, 1.8, n)
            elif value.dim() == 0:
                value = torch.tensor(rng.uniform(0.7, 1.5), dtype=torch.float32)
            elif key.endswith(".conv"):
                value = value * 1.5
            elif key == "loop.step":
                value = value * 25.0
            elif key == "bigram":
                value = value * 40.0
            elif key == "embed":
                value = value * (30.0 / raw["embedding"]["scale"])
            elif key.endswith((".mix.right.a", ".mix.right.b", ".mix.right.f")):
                value = value * 20.0
            elif key.endswith(".router"):
                value = value * 25.0
            elif ".mix." in key and value.dim() == 2:
                value = value * MIXER_SCALE[name] * (4.0 if key.endswith(".g") else 1.0)
            elif ".mlp.e" in key:
                value = value * EXPERT_SCALE[name]
            elif key == "head":
                value = value * 8.0
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
    write bfloat16, four times with a little noise before the rounding (nearly tied choices of experts fall either way): what
    rounding alone does at that place of that model."""
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
    """Every place that came back against the plain implementation, by the root mean square of the difference over the
    vocabulary divided by the logits' own spread there (``relative``); a failure names the first wrong token and what is
    special about its place.  ``rounded`` (16-bit runs): a place's bar is ``tol`` or, where the model is touchy, three times
    what rounding the plain implementation's matrix products does there; and four places in a hundred may be over it (a
    router's nearly tied choice may fall either way in 16 bits; the 32-bit run of the same plan has no such allowance)."""
    assert got, "no logits came back"
    worst, first, over, places = 0.0, None, 0, 0
    for rid, tokens in requests.items():
        want = plain_logits(directory, tokens)
        bars = np.maximum(tol, 3.0 * rounding_moves(directory, tokens)) if rounded else np.full(len(tokens), tol)
        for pos in range(len(tokens)):
            if (rid, pos) not in got:
                continue
            err = relative(got[(rid, pos)], want[pos])
            places += 1
            if not np.isfinite(err) or err > bars[pos]:
                over += 1
                if first is None:
                    first = (f"{label}: request {rid} position {pos} of {len(tokens)} (position % {page} = {pos % page}) "
                             f"differs by {err:.3e} > {bars[pos]:.3e}")
            worst = max(worst, err) if np.isfinite(err) else float("inf")
    if over > (max(2, 4 * places // 100) if rounded else 0) or not np.isfinite(worst):
        raise AssertionError(f"{first}; {over} of {places} places are over the bar")
    return worst
