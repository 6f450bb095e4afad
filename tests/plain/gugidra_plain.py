"""A plain, slow evaluation of the Gugidra decoder in float64, one function per mechanism, written from the design's
equations and sharing no code with the package.  A whole sequence at a time, no cache, no state carried: every
token's keys, values and recurrent state are recomputed from the layer's input.

Weights are a dict name -> torch tensor (any dtype; widened here), the configuration is the dict that
``config.json`` holds.  ``lowp=True`` rounds to bfloat16 where an engine's bfloat16 path may (operands and results of
matrix products, cached keys and values, the heads' outputs, experts' results); norms, angles, scores, softmax
weights, routers, decays, gates of a recurrence, the recurrences and the stream stay exact.  It measures what rounding
alone costs.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def _r(x, lowp):
    return x.to(torch.bfloat16).to(F64) if lowp else x


def product(x, w, lowp=False, bias=None):
    """x W^T (+ bias) for a weight stored [out, in]."""
    y = _r(x, lowp) @ w.to(F64).T
    if bias is not None:
        y = y + bias.to(F64)
    return _r(y, lowp)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_rms_norm(x, w, eps):
    """An RMS norm whose checkpoint weight is its gain less one."""
    return unit_rms(x, eps) * (1.0 + w.to(F64))


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------ linear attention with a decay per key channel
def channel_decay(h, w, prefix, tau, lowp=False):
    """log alpha [T, heads * dim], alpha = sigmoid(W_a2 W_a1 h + b)^(1 / tau)."""
    g = lambda n: w[prefix + n].to(F64)
    z = _r(_r(h, lowp) @ g("a1").T, False) @ g("a2").T + g("a2.b")
    return torch.nn.functional.logsigmoid(z) / tau


def gla_recurrence(q, k, v, alpha, S=None):
    """S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head; q, k, alpha [T, H, d], v [T, H, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if S is None else S.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, q[t])
    return out, S


def gla(h, w, prefix, m, eps, lowp=False):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    g = lambda n: w[prefix + n].to(F64)
    q = product(h, g("q"), lowp).view(T, H, d) * d ** -0.5
    k = product(h, g("k"), lowp).view(T, H, d)
    v = product(h, g("v"), lowp).view(T, H, dv)
    alpha = torch.exp(channel_decay(h, w, prefix, m["tau"], lowp)).view(T, H, d)
    o, _ = gla_recurrence(q, k, v, alpha)
    o = (unit_rms(o, eps) * g("norm")).reshape(T, H * dv) * silu(product(h, g("g"), lowp))
    return product(o, g("o"), lowp)


# ------------------------------------------------------------------ attention whose values are its unrotated keys
def turn_neighbours(x, base, dims):
    """Pairs (2i, 2i + 1) of the first ``dims`` entries turn by position * base^(-2i / dims); x [T, heads, d]."""
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=F64)
    for i in range(dims // 2):
        a = pos * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def key_value_attention(h, w, prefix, m, lowp=False):
    """Causal grouped-query attention; a token's value is its key as projected, before the rotation."""
    T, H, d = h.shape[0], m["heads"], m["dim"]
    G = m.get("kv_heads") or H
    g = lambda n: w[prefix + n].to(F64)
    q = product(h, g("q"), lowp, bias=g("q.b")).view(T, H, d)
    k = product(h, g("k"), lowp, bias=g("k.b")).view(T, G, d)
    v = k
    rot = m.get("rot")
    if rot:
        q, k = turn_neighbours(q, rot["base"], rot["dims"]), turn_neighbours(k, rot["base"], rot["dims"])
    q, k = _r(q, lowp), _r(k, lowp)
    seen = torch.arange(T)[:, None] >= torch.arange(T)[None, :]
    out = torch.zeros(T, H, d, dtype=F64)
    for n in range(H):
        s = ((q[:, n] @ k[:, n // (H // G)].T) * m["scale"]).masked_fill(~seen, -math.inf)
        out[:, n] = torch.softmax(s, dim=-1) @ v[:, n // (H // G)]
    return product(out.reshape(T, H * d), g("o"), lowp, bias=g("o.b"))


# ------------------------------------------------------------------ matrix memory
def memory_recurrence(q, k, v, i, f, state=None):
    """Per head, with log gates i and f [T, H] and a running maximum m: the state (S, n, m) and o_t."""
    T, H, d = q.shape
    dv = v.shape[-1]
    if state is None:
        state = (torch.zeros(H, d, dv, dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype), torch.zeros(H, dtype=q.dtype))
    S, n, m = (x.clone() for x in state)
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        m = m_new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hij,hi->hj", S, q[t]) / den[:, None]
    return out, (S, n, m)


def capped_gates(h, w, prefix, cap, lowp=False):
    """(i, f) [T, heads]: log input gate cap tanh(z / cap), log forget gate logsigmoid(cap tanh(z / cap))."""
    g = lambda n: w[prefix + n].to(F64)
    soft = lambda z: cap * torch.tanh(z / cap)
    hr = _r(h, lowp)
    return soft(hr @ g("i").T + g("i.b")), torch.nn.functional.logsigmoid(soft(hr @ g("f").T + g("f.b")))


def matrix_memory(h, w, prefix, m, eps, lowp=False):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    g = lambda n: w[prefix + n].to(F64)
    q = product(h, g("q"), lowp).view(T, H, d) * d ** -0.5
    k = product(h, g("k"), lowp).view(T, H, d)
    v = product(h, g("v"), lowp).view(T, H, dv)
    i, f = capped_gates(h, w, prefix, m["gate_cap"], lowp)
    o, _ = memory_recurrence(q, k, v, i, f)
    o = unit_rms(o, eps).reshape(T, H * dv) * g("norm") * torch.sigmoid(product(h, g("g"), lowp))
    return product(o, g("o"), lowp)


def side_by_side(h, w, prefix, m, eps, lowp=False):
    left = key_value_attention(h, w, prefix + "left.", m["left"], lowp)
    right = matrix_memory(h, w, prefix + "right.", m["right"], eps, lowp)
    return m["left_scale"] * left + m["right_scale"] * right


# ------------------------------------------------------------------ feed-forwards
def clamped_gate(g, u, limit):
    """g' sigmoid(1.702 g') (u' + 1) with g' = min(g, limit), u' = clamp(u, -limit, limit)."""
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def clamped_mlp(h, w, prefix, limit, lowp=False):
    a = clamped_gate(product(h, w[prefix + "gate"], lowp), product(h, w[prefix + "up"], lowp), limit)
    return product(a, w[prefix + "down"], lowp)


def choose(scores, correction, router):
    """The chosen experts per token, and (score gaps) how close each decision was."""
    choice = scores + correction
    E, top = choice.shape[-1], router["top"]
    groups = router.get("groups")
    gaps = []
    if groups and groups["count"] > 1:
        n, keep = groups["count"], groups["keep"]
        two = choice.view(-1, n, E // n).sort(-1, descending=True).values[..., :2].sum(-1)
        order = two.argsort(-1, descending=True)
        if keep < n:
            ranked = two.gather(-1, order)
            gaps.append(ranked[:, keep - 1] - ranked[:, keep])
        allowed = torch.zeros_like(two, dtype=torch.bool).scatter(-1, order[:, :keep], True)
        choice = choice.masked_fill(~allowed.repeat_interleave(E // n, dim=-1), -math.inf)
    ranked, idx = choice.sort(-1, descending=True)
    if top < E:
        gap = ranked[:, top - 1] - ranked[:, top]
        gaps.append(gap)
    return idx[:, :top], gaps


def routed_mlp(h, w, prefix, mlp, lowp=False, margins=None):
    router = mlp["router"]
    s = torch.sigmoid(_r(h, lowp) @ w[prefix + "router"].to(F64).T)
    idx, gaps = choose(s, w[prefix + "correction"].to(F64), router)
    if margins is not None and gaps:
        margins.extend(torch.stack(gaps).min(0).values.tolist())
    weight = s.gather(-1, idx)
    weight = weight / (weight.sum(-1, keepdim=True) + 1e-20)
    out = torch.zeros_like(h)
    for e in range(router["experts"]):
        tokens, place = torch.where(idx == e)
        if len(tokens):
            out[tokens] += weight[tokens, place, None] * clamped_mlp(h[tokens], w, f"{prefix}e{e}.", mlp["expert"]["limit"], lowp)
    if mlp.get("shared"):
        out = out + clamped_mlp(h, w, prefix + "shared.", mlp["shared"]["limit"], lowp)
    return out


# ------------------------------------------------------------------ the decoder
def layer_order(config):
    """(layer, pass that begins here or None) in the order the layers run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def forward(config, w, tokens, lowp=False, keep_layers=False, margins=None):
    """Logits [T, vocab] of one sequence from position 0 (and, with ``keep_layers``, the stream after every layer run)."""
    eps = float(config["norm"]["eps"])
    fed = w["embed"].to(F64)[torch.as_tensor(tokens, dtype=torch.long)] * float((config.get("embedding") or {}).get("scale", 1.0))
    x = fed
    kept = []
    for i, step in layer_order(config):
        L, p = config["layers"][i], f"l{i}."
        if step is not None:
            if step > 0:
                x = x + fed
            x = x + w["loop.step"].to(F64)[step]
        h = _r(centred_rms_norm(x, w[p + "norm1"], eps), lowp)
        mixer = {"gla": gla, "parallel": side_by_side}[L["type"]]
        x = x + centred_rms_norm(mixer(h, w, p + "mix.", L["mixer"], eps, lowp), w[p + "norm1b"], eps)
        mlp = L.get("mlp")
        if mlp:
            h = _r(centred_rms_norm(x, w[p + "norm2"], eps), lowp)
            if mlp["kind"] == "dense":
                f = clamped_mlp(h, w, p + "mlp.", mlp["limit"], lowp)
            else:
                f = routed_mlp(h, w, p + "mlp.", mlp, lowp, margins)
            x = x + centred_rms_norm(f, w[p + "norm2b"], eps)
        kept.append(x)
    logits = _r(centred_rms_norm(x, w["final.norm"], eps), lowp) @ w["head"].to(F64).T
    cap = config.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    return (logits, torch.stack(kept)) if keep_layers else logits
