"""Gugidra on the GPU: every new mechanism alone against the plain implementation's function for it, each mixer alone
through the package's cache manager and step context (batches of unequal entries, portions, slots and pages used again),
then the engine through the replay loop and through ``Engine.generate`` against the plain implementation of the whole
model, in 32-bit and in bfloat16, for four small configurations that differ in every size and option."""

import json
import math

import numpy as np
import pytest
import torch

import gugidra_helpers as GH
import helpers as H
from plain import gugidra_plain as GP

pytestmark = pytest.mark.gpu

BOTH = [torch.float32, torch.bfloat16]
F64 = torch.float64


@pytest.fixture(scope="module")
def ops():
    from pyre_b200.kernels import build, ops as o
    build.ensure_built(["matrix_state", "blockops", "grouped", "parallel_block", "elementwise", "gemm_tc", "gemm_f32"])
    return o


def close(got, want, dtype, what="", atol32=3e-6, rel16=1.6e-2):
    tol = dict(rtol=3e-5, atol=atol32) if dtype == torch.float32 else dict(rtol=rel16, atol=rel16)
    torch.testing.assert_close(got.double().cpu(), want.double().cpu(), msg=lambda m: f"{what}: {m}", **tol)


def bf16_exact(*shape, scale=1.0, seed=0):
    """Random fp64 values that bfloat16 holds exactly."""
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(torch.bfloat16).double()


# Sequences walked in steps of unequal portions (one token, a few, the sixteen of a block, more and less than a block, long
# ones beside single tokens), the last one starting later in the slot that the first one leaves: (sequence, tokens) per step.
SEQ_LENS = {"a": 9, "b": 171, "c": 67}
STEPS = [[("a", 1), ("b", 7)], [("a", 2), ("b", 1)], [("b", 33), ("a", 6)], [("b", 1)], [("b", 96), ("c", 1)], [("c", 32), ("b", 1)],
         [("c", 2)], [("b", 32), ("c", 1)], [("c", 31)]]
SLOT = {"a": 2, "b": 0, "c": 2}


def walk(seqs, launch):
    """Run ``launch(rows, slots, cu, lens) -> list of tensors [tokens, ...]`` over STEPS; the outputs per sequence."""
    at, out = {r: 0 for r in seqs}, {r: None for r in seqs}
    for step in STEPS:
        rows = torch.cat([torch.arange(seqs[r] + at[r], seqs[r] + at[r] + n) for r, n in step])
        lens = [n for _, n in step]
        cu = torch.tensor(np.concatenate([[0], np.cumsum(lens)]), dtype=torch.int32).cuda()
        slots = torch.tensor([SLOT[r] for r, _ in step], dtype=torch.int32).cuda()
        res = launch(rows.cuda(), slots, cu, lens, [r for r, _ in step if at[r] == 0])
        k = 0
        for r, n in step:
            new = [t[k:k + n].double().cpu() for t in res]
            out[r] = new if out[r] is None else [torch.cat([x, y]) for x, y in zip(out[r], new)]
            at[r], k = at[r] + n, k + n
    assert {r: at[r] for r in seqs} == SEQ_LENS
    return out


def starts():
    seqs, n = {}, 0
    for r, L in SEQ_LENS.items():
        seqs[r] = n
        n += L
    return seqs, n


# --------------------------------------------------------------------------- the recurrences, each alone
SIZES = [(3, 16, 24), (4, 20, 12), (2, 40, 16), (1, 128, 40), (4, 64, 128), (2, 48, 64), (1, 96, 8), (2, 33, 17), (1, 256, 32), (3, 8, 33)]


@pytest.mark.parametrize("dtype,chunked", [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)])
@pytest.mark.parametrize("heads,dk,dv", SIZES)
@pytest.mark.parametrize("strength", [0.2, 3.0, 60.0])
def test_decay_per_channel_recurrence(ops, dtype, chunked, heads, dk, dv, strength):
    """Token by token and in blocks of sixteen, over poisoned and reused slots, in columns of wider rows; decays from almost
    one to below exp(-100) within a block (where the blocks form every pair of tokens by itself)."""
    if strength != 0.2 and (heads, dk, dv) not in SIZES[:5]:
        return
    seqs, T = starts()
    W, off = 2 * heads * dk + heads * dv + 11, 3
    proj, z, bias = bf16_exact(T, W, seed=heads + dk), bf16_exact(T, heads * dk, scale=2.0, seed=dv), bf16_exact(heads * dk, seed=1)
    tau, qs = 1.0 / strength, dk ** -0.5
    state = torch.full((4, heads * dk * dv + 5), 7.0).cuda()
    pd, zd, bd = proj.to(dtype).cuda(), z.float().cuda(), bias.float().cuda()

    def launch(rows, slots, cu, lens, new):
        for r in new:
            state[SLOT[r]] = 0.0
            state[SLOT[r], heads * dk * dv:] = 7.0
        return [ops.gated_linear_attention(pd[rows].contiguous(), off, off + heads * dk, off + 2 * heads * dk, qs, zd[rows].contiguous(), bd, tau,
                                           state, slots, cu, heads, dk, dv, lens=lens, chunked=chunked)]
    got = walk(seqs, launch)
    for r, s in seqs.items():
        x = proj[s:s + SEQ_LENS[r]]
        q, k, v = (x[:, off + a:off + b].reshape(len(x), heads, -1) for a, b in ((0, heads * dk), (heads * dk, 2 * heads * dk),
                                                                              (2 * heads * dk, 2 * heads * dk + heads * dv)))
        alpha = torch.exp(torch.nn.functional.logsigmoid(z[s:s + SEQ_LENS[r]] + bias) / tau).view(len(x), heads, dk)
        want, _ = GP.gla_recurrence(q * qs, k, v, alpha)
        err, scale = (got[r][0].view_as(want) - want).abs(), float(want.abs().max())
        tol = 2e-5 if not chunked else 2e-4      # operands of the blocks carry 16 bits of mantissa
        assert float(err.max()) <= tol * scale, f"{r}: first wrong token {int(torch.where((err > tol * scale).flatten(1).any(1))[0][0])}, {float(err.max()) / scale:.2e}"
    assert (state[1] == 7.0).all() and (state[3] == 7.0).all() and (state[:, heads * dk * dv:] == 7.0).all(), "a slot that is not the step's, or beyond the state"


@pytest.mark.parametrize("dtype,chunked", [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)])
@pytest.mark.parametrize("heads,dk,dv", SIZES)
@pytest.mark.parametrize("cap,i_mean,f_mean", [(5.0, 0.0, 2.0), (12.0, -9.0, 8.0), (15.0, 6.0, -4.0)])
def test_matrix_memory_recurrence(ops, dtype, chunked, heads, dk, dv, cap, i_mean, f_mean):
    """o before the division and its denominator, with gates of order one, with inputs that are almost shut (the denominator
    is exp(-m) = 1 from the maximum's start at 0) and with inputs that grow while the memory forgets (the maximum moves on
    every token); gate logits as partial sums; the state's copies of the maximum agree afterwards."""
    if i_mean and (heads, dk, dv) not in SIZES[:5]:
        return
    seqs, T = starts()
    W, off = 2 * heads * dk + heads * dv + 13, 5
    proj = bf16_exact(T, W, seed=heads + dk)
    zi, zf = bf16_exact(T, heads, scale=3.0, seed=2) + i_mean, bf16_exact(T, heads, scale=3.0, seed=3) + f_mean
    bias = bf16_exact(2 * heads, seed=4)
    raw = torch.cat([zi, zf], dim=1)
    first = bf16_exact(T, 2 * heads, seed=5)
    parts = torch.stack([first, raw - first]).float().cuda()
    n = ops.memory_state_floats(heads, dk, dv)
    state = torch.full((4, n + 3), 7.0).cuda()
    pd, bd, qs = proj.to(dtype).cuda(), bias.float().cuda(), dk ** -0.5

    def launch(rows, slots, cu, lens, new):
        for r in new:
            state[SLOT[r], :n] = 0.0
        gates = ops.PartialSums(parts[:, rows].contiguous(), torch.float32)
        return list(ops.matrix_memory(pd[rows].contiguous(), off, off + heads * dk, off + 2 * heads * dk, qs, gates, bd, cap, state, slots, cu, heads,
                                      dk, dv, lens=lens, chunked=chunked))
    got = walk(seqs, launch)
    soft = lambda t: cap * torch.tanh(t / cap)
    for r, s in seqs.items():
        L = SEQ_LENS[r]
        x = proj[s:s + L]
        q, k, v = (x[:, off + a:off + b].reshape(L, heads, -1) for a, b in ((0, heads * dk), (heads * dk, 2 * heads * dk),
                                                                           (2 * heads * dk, 2 * heads * dk + heads * dv)))
        i = soft(zi[s:s + L] + bias[:heads])
        f = torch.nn.functional.logsigmoid(soft(zf[s:s + L] + bias[heads:]))
        want, (S, nn, m) = GP.memory_recurrence(q * qs, k, v, i, f)
        # the denominator by itself: a value of one per token, so that its numerator is n . q
        ones, _ = GP.memory_recurrence(q * qs, k, torch.ones(L, heads, 1, dtype=F64), i, f)
        mt, ms = torch.zeros(heads, dtype=F64), []
        for t in range(L):
            mt = torch.maximum(f[t] + mt, i[t])
            ms.append(mt)
        floor = torch.exp(-torch.stack(ms))
        den = got[r][1]
        # o / den = want, and the denominator is |n . q| or the floor, whichever is larger
        nq = (ones[..., 0] * den).abs()
        tol = 1e-4 if not chunked else 3e-4
        expect = torch.maximum(nq, floor) + 1e-6
        assert float(((den - expect).abs() / expect).max()) <= (1e-4 if not chunked else 2e-3), f"{r}: denominator"
        num = want * den[:, :, None]
        err, scale = (got[r][0].view_as(want) - num).abs(), num.abs().amax(dim=(1, 2), keepdim=True) + 1e-3 * num.abs().max()
        bad = (err > tol * scale).flatten(1).any(1)
        assert not bad.any(), f"{r}: first wrong token {int(torch.where(bad)[0][0])}, {float((err / scale).max()):.2e}"
        if r == "b":      # the state that the last step left
            st = state[SLOT[r]].double().cpu()
            base = heads * dk * dv
            assert float((st[base + heads * dk:n].view(heads, -1) - m[:, None]).abs().max()) <= 1e-4 * (1 + float(m.abs().max())), "copies of the maximum"
            assert float((st[base:base + heads * dk].view(heads, dk) - nn).abs().max()) <= 10 * tol * float(nn.abs().max()), "normaliser"
            assert float((st[:base].view(heads, dk, dv) - S).abs().max()) <= 10 * tol * float(S.abs().max()), "matrix"
    assert (state[1] == 7.0).all() and (state[:, n:] == 7.0).all()


@pytest.mark.parametrize("kind", ["decay", "memory"])
def test_a_token_by_token_result_does_not_depend_on_the_cut(ops, kind):
    """float32: the same bits whether the tokens come in one step, in portions or one by one beside others."""
    heads, dk, dv, T = 2, 48, 40, 61
    proj = torch.randn(T, 2 * heads * dk + heads * dv, generator=torch.Generator().manual_seed(0)).cuda()
    extra = torch.randn(T, max(heads * dk, 2 * heads), generator=torch.Generator().manual_seed(1)).cuda()
    bias = torch.zeros(heads * dk).cuda()

    def run(cuts):
        state, out, at = torch.zeros(2, ops.memory_state_floats(heads, dk, dv)).cuda(), [], 0
        for n in cuts:
            rows = slice(at, at + n)
            p, e, cu, slots = proj[rows].contiguous(), extra[rows], torch.tensor([0, n], dtype=torch.int32).cuda(), torch.zeros(1, dtype=torch.int32).cuda()
            if kind == "decay":
                out.append(ops.gated_linear_attention(p, 0, heads * dk, 2 * heads * dk, 0.2, e[:, :heads * dk].contiguous(), bias, 4.0, state, slots, cu, heads, dk, dv, lens=[n]))
            else:
                out.append(torch.cat(ops.matrix_memory(p, 0, heads * dk, 2 * heads * dk, 0.2, e[:, :2 * heads].contiguous(), bias[:2 * heads].contiguous(), 8.0, state,
                                                       slots, cu, heads, dk, dv, lens=[n]), dim=1))
            at += n
        return torch.cat(out)
    whole = run([T])
    assert torch.equal(whole, run([1] * T)) and torch.equal(whole, run([2, 17, 1, 16, 25]))


# --------------------------------------------------------------------------- the small kernels, each alone
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,dv,gate,per_head,with_den,post", [(3, 24, "silu", True, False, 1.0), (4, 36, "sigmoid", False, True, 0.7), (2, 128, "sigmoid", False, True, 1.3),
                                                                 (1, 7, "silu", True, True, 1.0), (5, 64, None, True, False, 2.0), (2, 300, "silu", False, False, 1.0)])
def test_heads_finish(ops, dtype, heads, dv, gate, per_head, with_den, post):
    T, W = 9, heads * dv
    o, den = bf16_exact(T, W, seed=1), bf16_exact(T, heads, seed=2).abs() + 0.25
    w = bf16_exact(dv if per_head else W, seed=3)
    proj = bf16_exact(T, W + 8, seed=4)
    out = torch.full((T, W + 12), 3.0, dtype=dtype).cuda()
    ops.heads_finish(o.float().cuda(), den.float().cuda() if with_den else None, w.float().cuda(), 1e-3, proj.to(dtype).cuda() if gate else None, 4, heads, dv,
                     dtype, gate=gate or "silu", post=post, out=out, out_col=8)
    u = o.view(T, heads, dv) / (den[:, :, None] if with_den else 1.0)
    want = (GP.unit_rms(u, 1e-3) * (w if per_head else w.view(heads, dv))).reshape(T, W) * post
    if gate:
        z = proj[:, 4:4 + W]
        want = want * (GP.silu(z) if gate == "silu" else torch.sigmoid(z))
    close(out[:, 8:8 + W], want, dtype, "heads")
    assert (out[:, :8] == 3.0).all() and (out[:, 8 + W:] == 3.0).all()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,I,limit", [(5, 72, 0.8), (3, 33, 2.0), (130, 256, 1.0), (300, 512, 0.5), (70, 128, 7.0)])
def test_clamped_gate_after_and_inside_the_product(ops, dtype, T, I, limit):
    Hn = 64
    x, wg, wu = bf16_exact(T, Hn, seed=T), bf16_exact(I, Hn, scale=0.3, seed=I), bf16_exact(I, Hn, scale=0.3, seed=I + 1)
    r = lambda t: t.to(torch.bfloat16).double() if dtype == torch.bfloat16 else t
    want = GP.clamped_gate(r(x @ wg.T), r(x @ wu.T), limit)
    assert (x @ wg.T > limit).any() and ((x @ wu.T).abs() > limit).any()
    stacked = torch.cat([wg, wu]).to(dtype).cuda()
    got = {"after": ops.act_mul(ops.materialize(ops.linear(x.to(dtype).cuda(), stacked)), "clamped", limit=limit),
           "stacked": ops.gated_linear(x.to(dtype).cuda(), stacked, False, kind="clamped", limit=limit)}
    if dtype == torch.bfloat16 and I % 128 == 0:
        w = ops.interleave_gate_up(wg.to(dtype).cuda(), wu.to(dtype).cuda())
        got["inside"] = ops.gated_linear(x.to(dtype).cuda(), w, True, kind="clamped", limit=limit)
        assert torch.equal(got["inside"], got["after"]), "the epilogue's activation is the kernel's"
    for what, g in got.items():
        close(g, want, dtype, what, atol32=1e-5)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("E,top,count,keep,shift", [(8, 3, 2, 1, 0.0), (9, 3, 3, 1, -1.5), (16, 4, 4, 2, -0.7), (6, 2, 6, 3, 0.0), (40, 5, 5, 2, 0.3), (64, 6, 8, 4, -2.0), (70, 4, 35, 9, 0.0)])
def test_router_of_groups(ops, dtype, E, top, count, keep, shift):
    """The best groups by the sum of their two largest choice scores, also where every choice score is negative; weights
    without the correction."""
    T, Hn = 13, 92
    h, w, c = bf16_exact(T, Hn, seed=E), bf16_exact(E, Hn, scale=0.2, seed=E + 1), bf16_exact(E, scale=0.3, seed=E + 2) + shift
    c = c.float().double()
    s = torch.sigmoid(h @ w.T)
    order, _ = GP.choose(s, c, {"top": top, "groups": {"count": count, "keep": keep}} if count < E else {"top": top})
    if count == E:      # groups of one: a group's score is its expert's
        order = (s + c).argsort(-1, descending=True)[:, :top]
    idx, wt = ops.route(h.to(dtype).cuda(), w.float().cuda(), c.float().cuda(), top, 1.0, sigmoid=True, renormalise=True, renorm_eps=1e-20, groups=count, keep=keep)
    assert torch.equal(idx.cpu().long(), order)
    picked = s.gather(-1, order)
    close(wt, picked / picked.sum(-1, keepdim=True), torch.float32, "weights", atol32=1e-5)
    free = (s + c).argsort(-1, descending=True)[:, :top]
    assert count == E or not torch.equal(free, order), "this case would not show groups that are ignored"


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("nh,nkv,dk,rot,D,pad", [(4, 2, 32, 16, 32, 0), (5, 5, 20, 12, 32, 3), (2, 1, 128, 128, 128, 8), (6, 1, 48, 0, 64, 4), (3, 3, 20, 20, 32, 1)])
def test_biases_and_values_that_are_the_unrotated_keys(ops, dtype, nh, nkv, dk, rot, D, pad):
    T, page = 7, 4
    W = (nh + nkv) * dk + 2 * pad
    proj, qb, kb = bf16_exact(T, W, seed=nh), bf16_exact(nh * dk, seed=1), bf16_exact(nkv * dk, seed=2)
    cache = torch.full((4, 2, nkv, page, D), 9.0, dtype=dtype).cuda()
    where = torch.tensor([3, 0, 7, 12, 1, -1, 15], dtype=torch.int32)
    pos = torch.tensor([0, 1, 2, 3, 4, 5, 6], dtype=torch.int32)
    cos = sin = None
    if rot:
        inv = (100.0 ** (-torch.arange(0, rot, 2, dtype=F64) / rot)).float().cuda()
        cos, sin = ops.rope_table(pos.cuda(), inv)
    q = ops.qk_norm_rope_write(proj.to(dtype).cuda(), pad, pad + nh * dk, pad + nh * dk, None, None, 0.0, cos, sin, cache, where.cuda(), nh, nkv, dk, dk, D,
                               rot, page, neighbours=True, biases=(qb.float().cuda(), kb.float().cuda(), kb.float().cuda()))
    rows = proj[:, pad:pad + (nh + nkv) * dk] + torch.cat([qb, kb])
    wq, wk = rows[:, :nh * dk].view(T, nh, dk), rows[:, nh * dk:].view(T, nkv, dk)
    turn = lambda t: GP.turn_neighbours(t, 100.0, rot)
    close(q.view(T, nh, D)[..., :dk], turn(wq), dtype, "queries", atol32=2e-5)
    assert (q.view(T, nh, D)[..., dk:] == 0).all()
    for t in range(T):
        if where[t] >= 0:
            p, o = divmod(int(where[t]), page)
            close(cache[p, 0, :, o, :dk], turn(wk)[t], dtype, "key", atol32=2e-5)
            close(cache[p, 1, :, o, :dk], wk[t], dtype, "value: the key before it turns", atol32=2e-5)
            assert (cache[p, :, :, o, dk:] == 0).all()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("Hn", [96, 92, 33, 2048, 4100, 3000])
@pytest.mark.parametrize("form", ["tensor", "parts", "biased"])
def test_norm_update_and_next_norm_in_one(ops, dtype, Hn, form):
    """The same as the two kernels behind one another, to rounding of the sums, on all rows and on gathered ones."""
    T, eps_b, eps = 6, 1e-3, 1e-5
    x, y, b = bf16_exact(T, Hn, seed=1), bf16_exact(T, Hn, seed=2), bf16_exact(Hn, seed=3)
    wb, w = bf16_exact(Hn, seed=4), bf16_exact(Hn, seed=5)
    if form == "parts":
        first = bf16_exact(T, Hn, seed=6)
        val = ops.PartialSums(torch.stack([first, y - first]).float().cuda(), dtype)
    else:
        val = y.to(dtype).cuda()
    if form == "biased":
        val = ops.BiasedRows(val, b.float().cuda())
    v = y + b if form == "biased" else y
    stream = x + GP.unit_rms(v, eps_b) * wb
    want = GP.unit_rms(stream, eps) * w
    xd = x.float().cuda()
    branch = ops.NormedBranch(val, wb.float().cuda(), eps_b, dtype)
    rows = torch.tensor([4, 1], dtype=torch.int32).cuda()
    close(ops.add_rmsnorm(xd, branch, w.float().cuda(), eps, dtype, rows=rows), want[[4, 1]], dtype, "gathered rows", atol32=2e-5)
    assert torch.equal(xd, x.float().cuda()), "gathering leaves the stream alone"
    close(ops.add_rmsnorm(xd, branch, w.float().cuda(), eps, dtype), want, dtype, "all rows", atol32=2e-5)
    close(xd, stream, torch.float32, "the stream", atol32=2e-5)
    formed = branch.formed()
    formed = formed.parts[0] if isinstance(formed, ops.PartialSums) else formed
    close(formed, stream - x, torch.float32, "formed for another consumer", atol32=2e-5)


@pytest.mark.parametrize("dtype", BOTH)
def test_heads_copied_beside_others(ops, dtype):
    T, nh, D, dv = 5, 3, 32, 20
    a = bf16_exact(T, nh * D, seed=1)
    out = torch.full((T, nh * dv + 16), 5.0, dtype=dtype).cuda()
    ops.sigmoid_gate(a.to(dtype).cuda(), D, None, -1, nh, dv, out=out, out_col=8, scale=0.6)
    close(out[:, 8:8 + nh * dv], (a.view(T, nh, D)[..., :dv] * 0.6).reshape(T, -1), dtype, "heads")
    assert (out[:, :8] == 5.0).all() and (out[:, 8 + nh * dv:] == 5.0).all()


# --------------------------------------------------------------------------- each mixer alone through the cache manager
def run_mixer_alone(tmp_path, layer, width, eps, dtype, page, steps, inputs, seed, edit=None):
    """A model of this one layer is loaded (registry, loader, cache and state groups as ever), and its MIXER is called
    with inputs of the test's own on the step contexts that the package's stepper builds for ``steps`` (lists of
    (request, tokens) per step; a request begins at its first entry and ends after its last).  Returns the mixer's
    rows per request and the weights."""
    from pyre_b200.engine.replay import runtime_for_model
    from pyre_b200.engine.step import StepEntry
    from pyre_b200.kernels import ops
    from pyre_b200.models.model import load_model
    from safetensors.torch import load_file
    raw = {"architecture": "Gugidra", "vocab": 32, "width": width, "norm": {"eps": eps}, "layers": [dict(layer, mlp=None)]}
    GH.make_gugidra_dir(tmp_path, raw, seed=seed, edit=edit)
    model, _ = load_model(tmp_path, "cuda", dtype)
    as_trace = [{"entries": [{"id": r, "tokens": [0] * n} for r, n in st],
                 "end": [r for r, _ in st if all(r != x for later in steps[i + 1:] for x, _ in later)]} for i, st in enumerate(steps)]
    cache, stepper = runtime_for_model(model, H.max_live_tokens(as_trace), page, max_requests=max(len(st) for st in steps), poison=True,
                                       cuda_graphs=False)
    mixer, call = model.blocks[0].mixer, model.calls[0]
    at, out = {}, {}
    for i, step in enumerate(steps):
        for r, _ in step:
            if r not in at:
                cache.begin(r)
                at[r], out[r] = 0, []
        ctx = stepper.build_context([StepEntry(r, [0] * n, []) for r, n in step])
        h = torch.cat([inputs[r][at[r]:at[r] + n] for r, n in step]).to(model.dtype).cuda()
        rows = ops.materialize(mixer.forward(ctx, h, call)).float().cpu()
        k = 0
        for (r, n), new_len in zip(step, ctx.new_lens):
            cache.commit(r, new_len)
            out[r].append(rows[k:k + n])
            at[r], k = at[r] + n, k + n
        later = {x for st in steps[i + 1:] for x, _ in st}
        for r, _ in step:
            if r not in later:
                cache.end(r)
    ops.check_device_errors()
    cache.check()
    assert not cache.live()
    return {r: torch.cat(v) for r, v in out.items()}, load_file(str(tmp_path / "model.safetensors"))


MIXER_LENGTHS = {"a": 1, "b": 2, "c": 50, "d": 33, "e": 130, "f": 17}


def mixer_schedule(lengths, seed):
    """Steps of up to three live requests: portions of 1 to 48 tokens until each request has had all of its tokens; six
    requests in all, so slots and pages are used again."""
    rng = np.random.default_rng(seed)
    waiting, live, left, steps = list(lengths.items()), [], {}, []
    while waiting or live:
        while waiting and len(live) < 3:
            r, n = waiting.pop(0)
            live.append(r)
            left[r] = n
        step = []
        for r in list(live):
            n = min(left[r], int(rng.choice([1, 1, 2, 5, 9, 32, 48])))
            step.append((r, n))
            left[r] -= n
            if not left[r]:
                live.remove(r)
        steps.append(step)
    return steps


def check_mixer(tmp_path, layer, width, eps, dtype, page, plain, seed, inputs=None, edit=None, wrong=None):
    inputs = inputs or {r: bf16_exact(n, width, seed=seed + i) for i, (r, n) in enumerate(MIXER_LENGTHS.items())}
    got, w = run_mixer_alone(tmp_path, layer, width, eps, dtype, page, mixer_schedule({r: len(h) for r, h in inputs.items()}, seed), inputs, seed, edit)
    for r, h in inputs.items():
        want = plain(h, w)
        err = (got[r].double() - want).abs()
        bound = (3e-5 if dtype == "float32" else 5e-2) * (1.0 + want.abs())
        bad = (err > bound).any(dim=1)
        assert not bad.any(), f"request {r}: first wrong token {int(torch.where(bad)[0][0])} of {h.shape[0]}, max error {float(err.max()):.3e}"
        if wrong is not None and r in wrong[1]:      # the test can see the fault it is there for
            assert ((wrong[0](h, w) - want).abs() > 2 * 5e-2 * (1.0 + want.abs())).any(), f"request {r} would not show the fault"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dk,dv,tau,rank,width", [(3, 16, 24, 8.0, 6, 96), (4, 20, 12, 3.0, 5, 92), (4, 64, 128, 16.0, 16, 256), (1, 128, 40, 1.0, 24, 128),
                                                        (2, 40, 16, 16.0, 12, 64), (1, 200, 32, 0.5, 3, 40)])
def test_gated_linear_attention_alone(tmp_path, dtype, heads, dk, dv, tau, rank, width):
    layer = GH.gla(heads, dk, dv, tau, rank)
    check_mixer(tmp_path, layer, width, 1e-5, dtype, 16, lambda h, w: GP.gla(h, w, "l0.mix.", layer["mixer"], 1e-5), seed=heads)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("left,right,scales,page,width", [
    ((4, 2, 32, 0.25, 16, 100.0), (3, 16, 24, 5.0), (0.7, 1.4), 16, 96), ((5, 5, 20, 0.3, 12, 500.0), (4, 12, 36, 15.0), (1.0, 1.0), 8, 92),
    ((8, 2, 64, 0.12, 64, 500000.0), (4, 64, 128, 12.0), (0.8, 0.9), 32, 256), ((6, 1, 48, 0.14, 0, 10000.0), (1, 96, 8, 10.0), (0.9, 0.3), 16, 128),
    ((4, 4, 128, 0.09, 32, 10000.0), (2, 128, 64, 20.0), (1.1, 0.6), 16, 256), ((2, 1, 16, 0.4, 16, 50.0), (2, 24, 40, 9.0), (1.0, 0.0), 4, 64),
    ((2, 2, 160, 0.08, 96, 10000.0), (1, 16, 16, 6.0), (0.0, 1.0), 16, 72)])
def test_attention_beside_a_matrix_memory_alone(tmp_path, dtype, left, right, scales, page, width):
    """Both branches together and, with a factor of zero on the other one, each by itself."""
    layer = GH.parallel(left, right, *scales)
    check_mixer(tmp_path, layer, width, 1e-5, dtype, page, lambda h, w: GP.side_by_side(h, w, "l0.mix.", layer["mixer"], 1e-5), seed=left[0])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H_,G,d,rot,page", [(2, 1, 32, 8, 16), (4, 2, 64, 16, 16), (1, 1, 128, 32, 8)])
def test_a_far_key_stands_out(tmp_path, dtype, H_, G, d, rot, page):
    """One early token whose key meets two late tokens' queries (one map makes the keys and, from the input's entries in
    another order, the queries; those tokens' inputs are the early one's in that order, large): its score stands out among
    hundreds, in a prompt's last portion and in a decoded token, so an attention that misses that key (on the first page, at
    a page's border) is far off."""
    width, n, turn = 64, 300, 29
    layer = GH.parallel((H_, G, d, d ** -0.5, rot, 1e6), (1, 8, 8, 6.0), 1.0, 0.0)

    def edit(state):
        k = state["l0.mix.left.k"].view(G, d, width)
        k[:, :rot] = 0.0                                                   # the match lies in the entries that do not turn
        state["l0.mix.left.q"] = torch.roll(k.repeat_interleave(H_ // G, dim=0).reshape(H_ * d, width), -turn, dims=1).clone()
        for nm in ("l0.mix.left.q.b", "l0.mix.left.k.b"):
            state[nm] = state[nm] * 0.1
    inputs = {}
    for i, (r, far) in enumerate((("first", 0), ("border", page - 1), ("next", page), ("later", 3 * page + 1))):
        h = bf16_exact(n - 37 * i, width, scale=0.3, seed=70 + i)
        h[far] = bf16_exact(width, scale=3.0, seed=80 + i)
        h[-1] = h[-20] = torch.roll(h[far], -turn)
        inputs[r] = h
    far_of = {len(h): f for (r, h), f in zip(inputs.items(), (0, page - 1, page, 3 * page + 1))}

    def plain(h, w, drop=False):
        if drop:      # the far token's key and value are those of a token like the others
            h = h.clone()
            h2 = h.clone()
            h2[far_of[len(h)]] = h[far_of[len(h)] + 1]
            last = GP.side_by_side(h2, w, "l0.mix.", layer["mixer"], 1e-5)
            return torch.cat([GP.side_by_side(h, w, "l0.mix.", layer["mixer"], 1e-5)[:-25], last[-25:]])
        return GP.side_by_side(h, w, "l0.mix.", layer["mixer"], 1e-5)
    check_mixer(tmp_path, layer, width, 1e-5, dtype, page, plain, seed=3, inputs=inputs, edit=edit, wrong=(lambda h, w: plain(h, w, True), list(inputs)))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,Hn,mlp", [(9, 96, GH.moe(32, 0.6, 6, 2, (3, 2), (40, 1.1))), (7, 92, GH.moe(20, 0.7, 3, 3)), (300, 256, GH.moe(128, 1.0, 8, 2, (4, 1), (256, 2.0))),
                                      (4, 128, GH.moe(64, 0.5, 1, 1, None, (64, 3.0))), (64, 64, GH.moe(24, 1.5, 9, 3, (3, 1), (24, 0.8)))])
def test_routed_feed_forward(ops, dtype, T, Hn, mlp):
    """Clamped experts of the best groups, renormalised weights, a shared expert with a limit of its own; inputs on which no
    decision is a close call."""
    from pyre_b200.parts.base import PartSpec, collect_tensors, load_part, make_part
    from pyre_b200.weights.loader import target_dtype
    g = torch.Generator().manual_seed(T)
    E, ff, shared = mlp["router"]["experts"], mlp["expert"]["ff"], mlp.get("shared")
    groups = mlp["router"].get("groups")
    part = make_part("ffn", PartSpec("routed_mlp", {"width": Hn, "intermediate": ff, "n_experts": E, "top": mlp["router"]["top"], "activation": "clamped",
                                                    "limit": mlp["expert"]["limit"], "scores": "sigmoid", "renormalise": True, "renorm_eps": 1e-20,
                                                    "groups": (groups["count"], groups["keep"]) if groups else None,
                                                    "shared": shared["ff"] if shared else None, "shared_limit": shared["limit"] if shared else None}), dtype, "cuda")
    specs = collect_tensors(part, "p.")
    w = {n: bf16_exact(*s.shape, scale=0.25 if len(s.shape) == 2 else 0.2, seed=i) for i, (n, s) in enumerate(specs.items())}
    rows = []
    while len(rows) < T:
        h = torch.randn(1, Hn, generator=g).to(torch.bfloat16).double()
        margins = []
        GP.routed_mlp(h, w, "p.", mlp, margins=margins)
        if not margins or margins[0] > 0.01:
            rows.append(h)
    h = torch.cat(rows)
    want = GP.routed_mlp(h, w, "p.", mlp)
    load_part(part, {n: w[n].to(target_dtype(s, torch.float32, dtype)).cuda() for n, s in specs.items()}, "p.")
    got = ops.materialize(part.forward(None, h.to(dtype).cuda())).float()
    bound = (2e-5 if dtype == torch.float32 else 3e-2) * float(want.abs().max())
    assert float((got.double().cpu() - want).abs().max()) <= bound


# --------------------------------------------------------------------------- the engine against the plain model
LENGTHS = {"A": [1, 2, 17, 33, 70, 130], "B": [5, 31, 97, 120], "C": [3, 63, 64, 65, 130], "D": [2, 47, 129]}
LONG = {"A": [160, 130], "C": [120, 100]}      # decoded one by one from token 70 (40) on


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for n, (name, raw) in enumerate(GH.GUG.items()):
        d = tmp_path_factory.mktemp(f"gugidra_{name}")
        GH.make_gugidra_dir(d, raw, seed=700 + n)
        reqs = {f"{name}{i}": GH.decided_ids(d, L, seed=13 * n + i) for i, L in enumerate(LENGTHS[name])}
        plain = {rid: GH.plain_logits(d, ids) for rid, ids in reqs.items()}
        lowp = {rid: GH.rounded_logits(d, ids, plain[rid]) for rid, ids in reqs.items()}
        sq = sum(float(((lowp[rid] - plain[rid]) ** 2).sum()) for rid in reqs)
        long_reqs = {f"long{i}": GH.decided_ids(d, L, seed=90 + i) for i, L in enumerate(LONG.get(name, []))}
        long_plain = {r: (p, GH.rounded_logits(d, long_reqs[r], p)) for r, p in ((r, GH.plain_logits(d, ids)) for r, ids in long_reqs.items())}
        out[name] = (d, reqs, plain, math.sqrt(sq / sum(p.size for p in plain.values())), lowp, long_reqs, long_plain)
    return out


def run(models, name, dtype, steps, what, rename=None):
    d, reqs, plain, lowp_rms, lowp = models[name][:5]
    got = H.run_trace_in_process(d, dtype, steps, H.max_live_tokens(steps), GH.GUG_PAGE_SIZE[name])
    if rename:
        plain, lowp = ({new: src[old] for new, old in rename.items()} for src in (plain, lowp))
    GH.compare(got, plain, dtype, what, lowp_rms, lowp)


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_the_stream_after_every_layer(models, name):
    """In 32-bit, the stream after each layer against the plain implementation's: the first layer that differs is named."""
    from pyre_b200.engine.replay import runtime_for_model
    from pyre_b200.engine.step import StepEntry
    from pyre_b200.kernels import ops
    from pyre_b200.models.model import load_model
    from safetensors.torch import load_file
    d, reqs = models[name][:2]
    ids = max(reqs.values(), key=len)[:48]
    with torch.inference_mode():
        _logits, want = GP.forward(GH.GUG[name], load_file(str(d / "model.safetensors")), ids, keep_layers=True)
    model, _ = load_model(d, "cuda", "float32")
    cache, stepper = runtime_for_model(model, 64, GH.GUG_PAGE_SIZE[name], max_requests=1, cuda_graphs=False)
    cache.begin("r")
    ctx = stepper.build_context([StepEntry("r", ids, [])])
    x, pending = model.embed.forward(ctx), None
    fed = x.clone()
    for n, call in enumerate(model.calls):
        if call.add_embedding:
            ops.add_residual(x, fed)
        if call.add_vector is not None:
            ops.add_row_vector(x, model.vectors[call.add_vector[0]][call.add_vector[1]])
        x, pending = model.blocks[call.block].forward(ctx, x, pending, call)
        now = x + ops.materialize(pending).float() if pending is not None else x
        err = (now.double().cpu() - want[n]).abs().max()
        assert err < 2e-4 * (1 + want[n].abs().max()), f"layer {call.block} ({GH.GUG[name]['layers'][call.block]['type']}): off by {float(err):.3e}"
    cache.end("r")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_whole_prompts(models, name, dtype):
    run(models, name, dtype, H.trace_whole(models[name][1]), "whole")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_prefill_then_token_by_token(models, name, dtype):
    steps = []
    for k, (rid, ids) in enumerate(models[name][1].items()):
        # most of it in one step and the rest one by one; every third request one by one from its first token
        steps += H.trace_decode_tail(rid, ids, len(ids) if k % 3 == 2 else 32, first_step=len(steps))
    run(models, name, dtype, steps, "decode")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_portions_down_to_two_tokens(models, name, dtype):
    steps = []
    for k, (rid, ids) in enumerate(models[name][1].items()):
        sizes = [[2, 9, 3, 17, 2, 31], [5, 2, 16, 8, 64], [24, 2, 2, 7, 1, 70]][k % 3]
        steps += H.trace_portions(rid, ids, sizes, first_step=len(steps))
    run(models, name, dtype, steps, "portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_mixed_batches_reuse_pages_and_slots(models, name, dtype):
    """Every request twice under other names, at most four alive: later ones get the pages (filled with NaN when they were
    given back) and the state slots that earlier ones held, and must come out as each alone."""
    reqs = models[name][1]
    many = {f"{rid}r{rep}": ids for rep in range(2) for rid, ids in reqs.items()}
    steps = H.trace_mixed(many, seed=21, max_live=4, portion=(2, 40))
    run(models, name, dtype, steps, "mixed", rename={f"{rid}r{rep}": rid for rep in range(2) for rid in reqs})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding(models, name, dtype):
    """Up to 160 tokens, the last 50 to 90 one by one (captured decode steps), two requests side by side: the recurrent
    states are carried through every step."""
    d, lowp_rms, reqs, long_plain = models[name][0], models[name][3], models[name][5], models[name][6]
    steps = [{"step": 0, "entries": [{"id": r, "tokens": ids[:70 - 30 * i], "want": [0]} for i, (r, ids) in enumerate(reqs.items())], "end": []}]
    at = {r: 70 - 30 * i for i, r in enumerate(reqs)}
    while any(at[r] < len(reqs[r]) for r in reqs):
        entries = [{"id": r, "tokens": [reqs[r][at[r]]], "want": [0]} for r in reqs if at[r] < len(reqs[r])]
        for e in entries:
            at[e["id"]] += 1
        steps.append({"step": len(steps), "entries": entries, "end": [e["id"] for e in entries if at[e["id"]] == len(reqs[e["id"]])]})
    got = H.run_trace_in_process(d, dtype, steps, H.max_live_tokens(steps), GH.GUG_PAGE_SIZE[name])
    want, lowp = {}, {}
    for i, r in enumerate(reqs):
        for dst, full in ((want, long_plain[r][0]), (lowp, long_plain[r][1])):
            dst[r] = np.concatenate([full[:1], full[70 - 30 * i:]])
    GH.compare(got, want, dtype, "long decoding", lowp_rms, lowp)


@pytest.mark.parametrize("name,seqs,pages", [("A", 3, 5), ("C", 3, 5), ("A", 6, 14)])
def test_greedy_generation_through_the_engine(models, name, seqs, pages):
    """``Engine.generate`` (scheduler, portions of prompts, captured decode steps, sampler) gives the tokens that
    the plain implementation's argmax gives, in 32-bit; a cache too small for all requests at once makes the
    scheduler preempt and recompute, state slots included; six requests side by side decode in captured steps that are
    padded with rows of no request (the scratch page and the scratch state slot)."""
    from pyre_b200.engine.engine import Engine
    from pyre_b200.sampling import SamplingParams
    d = models[name][0]
    raw = GH.GUG[name]
    prompts = [H.random_ids(raw["vocab"], n, seed=40 + n) for n in ((15, 16, 3, 30) if seqs == 3 else (15, 16, 3, 30, 7, 11))]
    new = 12
    engine = Engine(str(d), dtype="float32", page_size=16, num_pages=pages, max_num_seqs=seqs, max_num_batched_tokens=32, prefill_chunk=20)
    outs = engine.generate(prompts, SamplingParams(max_new_tokens=new, return_logits=True))
    for p, o in zip(prompts, outs):
        ids = list(p)
        for k in range(new):
            logits = GH.plain_logits(d, ids)[-1]
            top2 = np.sort(logits)[-2:]
            np.testing.assert_allclose(o.logits[k], logits, rtol=2e-4, atol=3e-5)
            if top2[1] - top2[0] > 1e-4:
                assert o.token_ids[k] == int(logits.argmax()), f"token {k} of a prompt of {len(p)}"
            ids.append(o.token_ids[k])
    assert json.dumps(engine.stats())
