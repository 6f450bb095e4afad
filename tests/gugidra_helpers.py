"""Fixtures of the Gugidra tests: small configurations that differ in every size and option, model folders with
random weights, and the plain implementation's logits."""

from __future__ import annotations

import json
from pathlib import Path

import numpy as np
import torch
from safetensors.torch import load_file, save_file

from plain import gugidra_plain
from tekarax_helpers import compare  # noqa: F401  (the same bounds serve: see its docstring)


def gla(heads, dim, vdim, tau, decay_rank):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": decay_rank}}


def parallel(left, right, left_scale, right_scale):
    """left: (heads, kv_heads, dim, scale, rot dims, base); right: (heads, dim, vdim, gate_cap)."""
    H, G, d, scale, rot, base = left
    m = {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": scale, "rot": {"dims": rot, "base": base}},
         "right": dict(zip(("heads", "dim", "vdim", "gate_cap"), right)), "left_scale": left_scale, "right_scale": right_scale}
    return {"type": "parallel", "mixer": m}


def with_mlp(layer, mlp=None):
    return dict(layer, mlp=mlp)


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff, limit, experts, top, groups=None, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


# The eps are large: a recurrent head whose sum nearly cancels is enlarged by its unit norm, the rounding in it with it, and
# with a small eps such a token says nothing about the engine in bfloat16.
# A: layers 1-2 run three times; a gla layer with wider values than keys, two of three groups of two experts; a layer without
#    a feed-forward; a rotation of half of each head; factors on both sides of one; a low gate cap; pages of 16.
GUG_A = {"architecture": "Gugidra", "vocab": 300, "width": 96, "norm": {"eps": 4e-3}, "embedding": {"scale": 3.0}, "logit_softcap": 1.5,
         "loop": {"start": 1, "stop": 3, "times": 3}, "layers": [
    with_mlp(parallel((4, 2, 32, 0.25, 16, 100.0), (3, 16, 24, 5.0), 0.7, 1.4), dense(160, 0.8)),
    with_mlp(gla(3, 16, 24, 8.0, 6), moe(32, 0.6, 6, 2, (3, 2), (40, 1.1))),
    with_mlp(parallel((2, 1, 16, 0.4, 16, 1000.0), (2, 24, 40, 9.0), 1.2, 0.5)),
    with_mlp(gla(2, 40, 16, 16.0, 12), dense(72, 2.5)),
]}
# B: no size is a multiple of 8 (width 92: the library product for odd K and the scalar paths), as many key/value heads as
#    query heads, a decay map of 5, keys wider than values and the other way round, no groups, no shared expert, all three
#    experts chosen, no repeated span, no cap on the logits; pages of 8.
GUG_B = {"architecture": "Gugidra", "vocab": 333, "width": 92, "norm": {"eps": 4e-2}, "layers": [
    with_mlp(gla(4, 20, 12, 3.0, 5), moe(20, 0.7, 3, 3)),
    with_mlp(parallel((5, 5, 20, 0.3, 12, 500.0), (4, 12, 36, 15.0), 1.0, 1.0), dense(66, 1.3)),
    with_mlp(gla(3, 12, 44, 1.0, 9)),
    with_mlp(parallel((6, 3, 20, 0.25, 20, 50.0), (3, 28, 12, 7.0), 0.4, 2.0), moe(28, 0.9, 4, 1, None, (20, 0.5))),
]}
# C: sizes of the tensor-core paths: attention heads of 64 and 128, memory heads of 64 x 128 and 128 x 64, gla heads of
#    64 x 128, feed-forwards wide enough for the fused products, four groups of which one is kept, the first layer twice.
GUG_C = {"architecture": "Gugidra", "vocab": 512, "width": 256, "norm": {"eps": 2e-2}, "embedding": {"scale": 16.0}, "logit_softcap": 40.0,
         "loop": {"start": 0, "stop": 1, "times": 2}, "layers": [
    with_mlp(parallel((8, 2, 64, 0.12, 64, 500000.0), (4, 64, 128, 12.0), 0.8, 0.9), moe(128, 1.0, 8, 2, (4, 1), (256, 2.0))),
    with_mlp(gla(4, 64, 128, 16.0, 16), dense(512, 1.5)),
    with_mlp(parallel((4, 4, 128, 0.09, 32, 10000.0), (2, 128, 64, 20.0), 1.1, 0.6), moe(128, 1.0, 16, 4, (4, 2))),
]}
# D: one head everywhere it can be one, keys of 128 with values of 40 and of 96 with values of 8, one expert of which one is
#    chosen, an inner size of 24, the whole stack twice, no rotation of one layer's heads.
GUG_D = {"architecture": "Gugidra", "vocab": 256, "width": 128, "norm": {"eps": 1.5e-2}, "embedding": {"scale": 0.5}, "logit_softcap": 25.0,
         "loop": {"start": 0, "stop": 3, "times": 2}, "layers": [
    with_mlp(gla(1, 128, 40, 30.0, 24), moe(64, 0.5, 1, 1, None, (64, 3.0))),
    with_mlp(parallel((6, 1, 48, 0.14, 0, 10000.0), (1, 96, 8, 10.0), 0.9, 0.3), dense(128, 0.4)),
    with_mlp(gla(5, 32, 32, 6.0, 8), moe(32, 1.5, 9, 3, (3, 1), (24, 0.8))),
]}
GUG = {"A": GUG_A, "B": GUG_B, "C": GUG_C, "D": GUG_D}
GUG_PAGE_SIZE = {"A": 16, "B": 8, "C": 32, "D": 16}
ROUTER_MARGIN = 1.2e-2     # a router decision closer than this could fall either way under bfloat16 rounding of the stream


def make_gugidra_dir(path: Path, raw: dict, seed: int, sharpen: float = 4.0, matrix_scale: float = 2.0, edit=None) -> dict:
    """config.json + model.safetensors (fp32 values that bfloat16 holds exactly) from the package's random mode.  The maps that
    make the attention's queries and keys are scaled up so that it is peaked, the recurrences' gates and decays, the
    biases, the corrections and the vectors of the repeated span so that each of them shows, the router so that its scores
    differ without saturating.  ``edit(state)`` changes tensors before they are rounded and written."""
    from pyre_b200.config import config_from_dict
    from pyre_b200.weights import random_state

    path.mkdir(parents=True, exist_ok=True)
    state = random_state(config_from_dict(raw), seed)
    for name, t in state.items():
        if name.endswith(("left.q", "left.k")):
            f = sharpen
        elif name.endswith(("left.q.b", "left.k.b", "left.o.b")):
            f = 15.0
        elif name.endswith(("right.i", "right.f")):
            f = 10.0
        elif name.endswith(".mlp.router"):
            f = 30.0 / raw["width"] ** 0.5
        elif name.endswith(".mlp.correction"):
            f = 8.0
        elif name.endswith(("mlp.gate", "mlp.up")) or ".gate" in name or ".up" in name:
            f = 5.0             # pre-activations that reach the limit
        elif name == "loop.step":
            f = 6.0
        else:
            f = matrix_scale if t.dim() == 2 and not name.endswith(".a2") else 1.0
        state[name] = t * f
    if edit is not None:
        edit(state)
    state = {k: v.to(torch.bfloat16).to(torch.float32).contiguous() for k, v in state.items()}
    (path / "config.json").write_text(json.dumps(raw))
    save_file(state, str(path / "model.safetensors"))
    return state


def decided_ids(path: Path, length: int, seed: int, chunk: int = 6) -> list:
    """Random token ids on which no router decision (of groups or of experts) is a close call: grown a few tokens at a time,
    a piece drawn again while any decision at its positions is closer than ROUTER_MARGIN (a decision depends on the tokens
    up to its own only)."""
    raw = json.loads((Path(path) / "config.json").read_text())
    rng = np.random.default_rng(seed)
    w = load_file(str(Path(path) / "model.safetensors"))
    ids: list = []
    while len(ids) < length:
        n = min(chunk, length - len(ids))
        best = None
        for _ in range(60):
            piece = [int(x) for x in rng.integers(0, raw["vocab"], n)]
            margins: list = []
            with torch.inference_mode():
                gugidra_plain.forward(raw, w, ids + piece, margins=margins)
            per_run = np.asarray(margins).reshape(-1, len(ids) + n)[:, -n:]       # one row per run of a routed layer that has a choice
            margin = float(per_run.min()) if per_run.size else 1.0
            if best is None or margin > best[0]:
                best = (margin, piece)
            if margin > ROUTER_MARGIN:
                break
        assert best[0] > ROUTER_MARGIN / 4, "no piece of tokens gave decided router choices"
        ids += best[1]
    return ids


def plain_logits(path: Path, ids, lowp: bool = False) -> np.ndarray:
    raw = json.loads((Path(path) / "config.json").read_text())
    w = load_file(str(Path(path) / "model.safetensors"))
    with torch.inference_mode():
        return gugidra_plain.forward(raw, w, list(ids), lowp=lowp).numpy()


def rounded_logits(path: Path, ids, plain: np.ndarray, variants: int = 4) -> np.ndarray:
    """What rounding can do at each position: of several evaluations rounded to bfloat16 where an engine may round (one as it
    is, the others with every matrix off by less than another such rounding) the row that is furthest from ``plain``.  A
    recurrent head whose sum nearly cancels is enlarged by its unit norm, so at such a token one evaluation says little
    about another one's error."""
    raw = json.loads((Path(path) / "config.json").read_text())
    w = load_file(str(Path(path) / "model.safetensors"))
    worst = None
    for v in range(variants):
        g = torch.Generator().manual_seed(v)
        near = w if v == 0 else {k: t * (1 + torch.randn(t.shape, generator=g) * 2.0 ** -9) if t.dim() == 2 else t for k, t in w.items()}
        with torch.inference_mode():
            got = gugidra_plain.forward(raw, near, list(ids), lowp=True).numpy()
        if worst is None:
            worst = got
        else:
            take = np.abs(got - plain).max(axis=1) > np.abs(worst - plain).max(axis=1)
            worst[take] = got[take]
    return worst
