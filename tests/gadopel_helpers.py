"""Fixtures of the Gadopel tests: small configurations that differ in every size and option, model folders with
random weights, and the plain implementation's logits."""

from __future__ import annotations

import json
from pathlib import Path

import numpy as np
import torch
from safetensors.torch import load_file, save_file

from plain import gadopel_plain
from tekarax_helpers import compare  # noqa: F401  (the same bounds serve: see its docstring)


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": scale, "rot": {"dims": rot_dim, "base": base}}}


def attn(heads, kv_heads, dim, vdim, scale, window, keep, rot_dims, base=10000.0, scaling=None):
    rot = {"dims": rot_dims, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": window, "keep_first": keep}, "rot": rot}}


def with_ff(layer, ff=0):
    return dict(layer, mlp={"kind": "dense", "ff": ff} if ff else None)


# A: a span in the middle that runs three times (layers 1-2); three key/value heads under six query heads, value heads
#    wider and smaller than key heads; part of a head rotated; a window of 11 beside 3 kept tokens and one of 29
#    beside 18 (more than a page of 16), so two cache groups of keys and values; layers without a feed-forward.
GAD_A = {"architecture": "Gadopel", "vocab": 300, "width": 96, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 3}, "layers": [
    with_ff(attn(6, 3, 16, 24, 0.3, 11, 3, 8, 100.0, (8.0, 32, 4.0, 1.0)), 160),
    with_ff(latent(3, 16, 8, 24, 40, 0.2), 96),
    with_ff(attn(4, 2, 32, 16, 0.2, 29, 18, 32, 1000.0, (3.0, 64, 8.0, 0.5))),
    with_ff(latent(5, 24, 16, 32, 16, 0.15, 500.0)),
]}
# B: no size is a multiple of 8 (width 92: the library product for odd K and the scalar paths; the exact latent kernel
#    in 32-bit, rows padded in 16-bit); as many key/value heads as query heads; no stretched frequencies; a window without
#    kept tokens, one with a single kept token, on pages of 8; no repeated span.
GAD_B = {"architecture": "Gadopel", "vocab": 333, "width": 92, "norm": {"eps": 3e-6}, "layers": [
    with_ff(latent(5, 20, 12, 12, 36, 0.18, 50.0), 66),
    with_ff(attn(5, 5, 20, 28, 0.25, 7, 1, 12, 50.0), 28),
    with_ff(attn(3, 3, 12, 12, 0.35, 9, 0, 12)),
    with_ff(latent(2, 28, 4, 40, 52, 0.3), 20),
]}
# C: sizes of the tensor-core paths: heads of 64 and 128 (the prompt kernels), a latent of 192 (two column groups), windows
#    of 64 beside 20 kept tokens and of 100 beside 70 (more than a key tile of 64) on pages of 32, feed-forwards wide
#    enough for the fused gated product; the first two layers twice.
GAD_C = {"architecture": "Gadopel", "vocab": 640, "width": 256, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 2, "times": 2}, "layers": [
    with_ff(attn(4, 2, 64, 48, 0.1, 64, 20, 64, 1000000.0, (4.0, 256, 32.0, 1.0)), 512),
    with_ff(latent(8, 64, 32, 64, 192, 0.09, 1000000.0), 256),
    with_ff(attn(4, 1, 128, 128, 0.05, 100, 70, 96, 10000.0, (2.0, 128, 16.0, 2.0)), 128),
]}
# D: more heads than a row tile of the latent kernel takes (72 > 64); six query heads over one key/value head with heads
#    of 48; a window wider than any request; a span of one layer that runs once.
GAD_D = {"architecture": "Gadopel", "vocab": 256, "width": 128, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 2, "times": 1}, "layers": [
    with_ff(latent(72, 16, 16, 8, 64, 0.2), 128),
    with_ff(attn(6, 1, 48, 40, 0.12, 100000, 5, 16, 10000.0, (2.0, 64, 8.0, 0.5)), 96),
]}
GAD = {"A": GAD_A, "B": GAD_B, "C": GAD_C, "D": GAD_D}
GAD_PAGE_SIZE = {"A": 16, "B": 8, "C": 32, "D": 16}


def make_gadopel_dir(path: Path, raw: dict, seed: int, sharpen: float = 5.0, matrix_scale: float = 2.0) -> dict:
    """config.json + model.safetensors (fp32 values that bfloat16 holds exactly) from the package's random mode.  The
    maps that make queries and keys are scaled up so that attention is peaked (with small random weights every score
    is near zero and a wrong key would change nothing); the pass's input matrix so that it keeps the stream's size."""
    from pyre_b200.config import config_from_dict
    from pyre_b200.weights import random_state

    path.mkdir(parents=True, exist_ok=True)
    state = random_state(config_from_dict(raw), seed)
    for name in state:
        if name.endswith((".mix.q", ".mix.k", ".mix.dkv", ".mix.uk")):
            state[name] = state[name] * sharpen
        elif name == "loop.in":
            state[name] = state[name] * (1.0 / (2.0 * raw["width"]) ** 0.5 / float(state[name].std()))
        elif state[name].dim() == 2:
            state[name] = state[name] * matrix_scale
        state[name] = state[name].to(torch.bfloat16).to(torch.float32)
    (path / "config.json").write_text(json.dumps(raw))
    save_file({k: v.contiguous() for k, v in state.items()}, str(path / "model.safetensors"))
    return state


def random_ids(raw: dict, n: int, seed: int) -> list:
    return [int(x) for x in np.random.default_rng(seed).integers(0, raw["vocab"], n)]


def plain_logits(path: Path, ids, lowp: bool = False) -> np.ndarray:
    raw = json.loads((Path(path) / "config.json").read_text())
    w = load_file(str(Path(path) / "model.safetensors"))
    with torch.inference_mode():
        return gadopel_plain.forward(list(ids), w, raw, lowp=lowp).numpy()
