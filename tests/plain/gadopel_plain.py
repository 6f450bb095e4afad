"""A plain, slow evaluation of the Gadopel decoder in float64, one function per mechanism, written from the design's
equations and sharing no code with the package.  A whole sequence at a time, no cache: every token's keys and values
are recomputed from the layer's input.

Weights are a dict name -> torch tensor (any dtype; widened here), the configuration is the dict that ``config.json``
holds.  ``lowp=True`` rounds to bfloat16 where an engine's bfloat16 path may (operands and results of matrix products,
the cached rows, the queries, the heads' outputs, activations); norms, angles, scores, the softmax and the stream stay
exact.  It measures what rounding alone costs.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def _r(x, lowp):
    return x.to(torch.bfloat16).to(F64) if lowp else x


def matmul(x, w, lowp=False, keep=False):
    """x W^T for a weight stored [out, in]; ``keep``: the result is not rounded (a product that enters the stream)."""
    y = _r(x, lowp) @ w.to(F64).T
    return y if keep else _r(y, lowp)


def layer_norm(x, gain, eps):
    """(x - mean) / sqrt(var + eps) * gain over the last axis; var is the mean squared deviation; no bias."""
    dev = x - x.mean(-1, keepdim=True)
    return dev / torch.sqrt((dev * dev).mean(-1, keepdim=True) + eps) * gain


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def frequencies(base, dims, scaling=None):
    """(pair frequencies, amplitude).  ``scaling`` {factor, original, fast, slow}: a ramp over the pair index between
    the pairs that turn ``fast`` and ``slow`` times within ``original`` positions decides how much of a frequency is
    divided by ``factor``; the amplitude is 0.1 ln(factor) + 1."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    fac, orig = float(scaling["factor"]), float(scaling["original"])

    def index(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(index(scaling["fast"])), 0)
    hi = min(math.ceil(index(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / fac * r + fi * (1.0 - r))
    return out, 0.1 * math.log(fac) + 1.0


def rotate(v, positions, base, dims, layout, scaling=None):
    """Entries of the leading ``dims`` turn in pairs: (i, i + dims / 2) for ``layout`` "half", (2i, 2i + 1) for
    "neighbours"; pair i by the angle position * frequency_i.  ``v`` [T, ..., n], ``positions`` [T]."""
    out = v.clone()
    freq, amp = frequencies(base, dims, scaling)
    shape = [v.shape[0]] + [1] * (v.dim() - 2)
    for i, f in enumerate(freq):
        a, b = (i, i + dims // 2) if layout == "half" else (2 * i, 2 * i + 1)
        ang = positions.to(F64) * f
        c, s = (torch.cos(ang) * amp).view(shape), (torch.sin(ang) * amp).view(shape)
        out[..., a] = v[..., a] * c - v[..., b] * s
        out[..., b] = v[..., b] * c + v[..., a] * s
    return out


def visible(T, window=None, keep_first=0):
    """seen[i, j]: j is not after i, and within the window of i or among the first ``keep_first``."""
    i, j = torch.arange(T).view(-1, 1), torch.arange(T).view(1, -1)
    seen = j <= i
    if window:
        seen = seen & ((i - j < window) | (j < keep_first))
    return seen


def softmax_sink(scores, seen, sink=None):
    """Weights over the visible keys; ``sink`` [H]: exp(sink) joins each denominator.  ``scores`` [H, T, T]."""
    s = scores.masked_fill(~seen, float("-inf"))
    m = s.amax(-1, keepdim=True)
    if sink is not None:
        m = torch.maximum(m, sink.view(-1, 1, 1))
    e = torch.exp(s - m)
    d = e.sum(-1, keepdim=True)
    if sink is not None:
        d = d + torch.exp(sink.view(-1, 1, 1) - m)
    return e / d


def latent_attention(h, w, pre, mx, eps, lowp=False):
    """Keys and values expanded per head from one cached latent per token, one rotated key part for all heads, a sink
    per head, one gate per head.  ``h`` [T, width] is one sequence from position 0."""
    T, H, dn, dr, dv, rank = h.shape[0], mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    g = lambda n: w[pre + n].to(F64)
    pos, rot = torch.arange(T), mx["rot"]
    q = matmul(h, g("q"), lowp).view(T, H, dn + dr)
    q_rot = _r(rotate(q[..., dn:], pos, rot["base"], rot["dims"], "half"), lowp)
    down = matmul(h, g("dkv"), lowp)
    c = _r(unit_rms(down[:, :rank], eps) * g("dkv.norm"), lowp)
    k_rot = _r(rotate(down[:, rank:], pos, rot["base"], rot["dims"], "half"), lowp)
    k = matmul(c, g("uk"), lowp).view(T, H, dn)
    v = matmul(c, g("uv"), lowp).view(T, H, dv)
    s = (torch.einsum("ihd,jhd->hij", q[..., :dn], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * mx["scale"]
    p = softmax_sink(s, visible(T), g("sink"))
    o = _r(torch.einsum("hij,jhd->ihd", p, v), lowp)
    o = _r(o * torch.sigmoid(matmul(h, g("g"), lowp)).unsqueeze(-1), lowp)
    return matmul(o.reshape(T, H * dv), g("o"), lowp)


def attention(h, w, pre, mx, eps, lowp=False):
    """Grouped-query attention: rotation of neighbouring pairs with scaled frequencies, then unit root mean square per
    head, a sliding window beside the first kept tokens, a plain softmax."""
    T, H, G, d, dv = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    g = lambda n: w[pre + n].to(F64)
    pos, rot, mask = torch.arange(T), mx["rot"], mx.get("mask") or {}

    def turned(name, heads):
        z = matmul(h, g(name), lowp).view(T, heads, d)
        return _r(unit_rms(rotate(z, pos, rot["base"], rot["dims"], "neighbours", rot.get("scaling")), eps), lowp)
    q, k = turned("q", H), turned("k", G).repeat_interleave(H // G, dim=1)
    v = matmul(h, g("v"), lowp).view(T, G, dv).repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * mx["scale"]
    p = softmax_sink(s, visible(T, mask.get("size"), mask.get("keep_first") or 0))
    o = _r(torch.einsum("hij,jhd->ihd", p, v), lowp)
    return matmul(o.reshape(T, H * dv), g("o"), lowp)


def feed_forward(h, w, pre, lowp=False):
    """W_down (relu(W_gate h) * (W_up h))."""
    g = lambda n: w[pre + n].to(F64)
    return matmul(_r(torch.relu(matmul(h, g("gate"), lowp)) * matmul(h, g("up"), lowp), lowp), g("down"), lowp)


def layer(x, w, i, cfg, lowp=False):
    """x + (mixer(norm1(x)) + ff(norm2(x))), both norms of the same x."""
    L, eps, pre = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    h = _r(layer_norm(x, w[pre + "norm1"].to(F64), eps), lowp)
    mix = {"latent_attention": latent_attention, "attention": attention}[L["type"]]
    add = mix(h, w, pre + "mix.", L["mixer"], eps, lowp)
    if L.get("mlp"):
        add = add + feed_forward(_r(layer_norm(x, w[pre + "norm2"].to(F64), eps), lowp), w, pre + "mlp.", lowp)
    return x + add


def feed_again(x, x0, w_in, lowp=False):
    """The stream at the start of a pass: W_in [x; x0]."""
    return matmul(torch.cat([x, x0], dim=-1), w_in, lowp, keep=True)


def layer_order(cfg):
    """(layer index, does a pass of the repeated span begin here?) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    order = [(i, False) for i in range(loop["start"])]
    for _ in range(loop["times"]):
        order += [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], n)]


def forward(tokens, w, cfg, streams=None, lowp=False):
    """Logits [T, vocab] (float64) of one sequence; ``streams``: a list that receives the stream after every layer run."""
    x0 = x = w["embed"].to(F64)[torch.as_tensor(tokens)]
    for i, begins in layer_order(cfg):
        if begins:
            x = feed_again(x, x0, w["loop.in"].to(F64), lowp)
        x = layer(x, w, i, cfg, lowp)
        if streams is not None:
            streams.append(x)
    return _r(layer_norm(x, w["final.norm"].to(F64), cfg["norm"]["eps"]), lowp) @ w["head"].to(F64).T
