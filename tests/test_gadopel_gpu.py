"""Gadopel on the GPU: every new mechanism alone against the plain implementation's function for it (windows beside kept
first tokens in every attention kernel, sinks and gates in every latent kernel, both rotations, the norm after the
rotation, two norms in one pass, the relu gate in every form of the gated product, the stream fed with the embedding
again), each mixer alone through the package's cache manager and step context, then the engine through the replay loop
and through ``Engine.generate`` against the plain implementation of the whole model, in 32-bit and in bfloat16, for four
small configurations that differ in every size and option."""

import json
import math

import numpy as np
import pytest
import torch

import gadopel_helpers as GH
import helpers as H
from plain import gadopel_plain as GP

pytestmark = pytest.mark.gpu

BOTH = [torch.float32, torch.bfloat16]
F64 = torch.float64


@pytest.fixture(scope="module")
def ops():
    from pyre_b200.kernels import ops as o
    return o


def close(got, want, dtype, what="", atol32=3e-6, rel16=1.6e-2):
    tol = dict(rtol=3e-5, atol=atol32) if dtype == torch.float32 else dict(rtol=rel16, atol=rel16)
    torch.testing.assert_close(got.double().cpu(), want.double().cpu(), msg=lambda m: f"{what}: {m}", **tol)


def bf16_exact(*shape, scale=1.0, seed=0):
    """Random fp64 values that bfloat16 holds exactly."""
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(torch.bfloat16).double()


def tables(ops, positions, base, dims, scaling=None):
    freq, amp = GP.frequencies(base, dims, scaling)
    cos, sin = ops.rope_table(positions.int().cuda(), torch.tensor(freq, dtype=F64).float().cuda())
    return cos * amp, sin * amp


# --------------------------------------------------------------------------- the small kernels, each alone
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,Hn,two", [(1, 96, True), (5, 92, False), (37, 1024, True), (3, 4100, True)])
def test_two_norms_of_one_stream_in_one_pass(ops, dtype, T, Hn, two):
    x = bf16_exact(T, Hn, seed=1) + 0.3
    a, f = bf16_exact(T, Hn, seed=2), bf16_exact(3, T, Hn, seed=3)      # a branch tensor, and a split product's parts
    ones = torch.ones(Hn, device="cuda")
    w1, w2 = (bf16_exact(Hn, seed=s).float() for s in (5, 6))
    want = x + a + (f.sum(0) if two else 0)
    xd = x.float().cuda()
    terms = [(a.to(dtype).cuda(), ones)] + ([(ops.PartialSums(f.float().cuda(), dtype), ones)] if two else [])
    h1, h2 = ops.add_layernorm(xd, ops.ScaledSum(terms, dtype), w1.cuda(), 1e-5, dtype, weight2=w2.cuda())
    close(xd, want, torch.float32, "stream", atol32=2e-5)
    close(h1, GP.layer_norm(want, w1.double(), 1e-5), dtype, "first norm", atol32=2e-5)
    close(h2, GP.layer_norm(want, w2.double(), 1e-5), dtype, "second norm", atol32=2e-5)
    # the second norm changes nothing of the first
    assert torch.equal(h1, ops.add_layernorm(xd.clone(), None, w1.cuda(), 1e-5, dtype))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,K,I", [(1, 96, 64), (3, 92, 50), (8, 256, 128), (40, 320, 384), (128, 256, 256), (200, 256, 384), (300, 512, 640), (2, 64, 20)])
def test_the_relu_gate_in_every_form_of_the_gated_product(ops, dtype, T, K, I):
    """Interleaved weights (the product's epilogue in both orientations, or the activation kernel where the plan does
    not fuse), stacked weights, and the separate kernel; negative gates give exact zeros."""
    x, gate, up = bf16_exact(T, K, seed=1), bf16_exact(I, K, scale=0.2, seed=2), bf16_exact(I, K, scale=0.2, seed=3)
    z, v = x @ gate.T, x @ up.T
    want = torch.relu(z) * v
    stacked = torch.cat([gate, up]).to(dtype).cuda()
    forms = {"stacked": ops.gated_linear(x.to(dtype).cuda(), stacked, False, kind="relu"),
             "kernel": ops.act_mul(ops.materialize(ops.linear(x.to(dtype).cuda(), stacked)), "relu")}
    if dtype == torch.bfloat16 and I % 128 == 0:
        woven = ops.interleave_gate_up(gate.to(dtype).cuda(), up.to(dtype).cuda())
        forms["woven"] = ops.gated_linear(x.to(dtype).cuda(), woven, True, kind="relu")
    bound = (2e-5 if dtype == torch.float32 else 2e-2) * (float(want.abs().max()) + 1.0)
    for name, got in forms.items():
        assert got.shape == (T, I)
        assert float((got.double().cpu() - want).abs().max()) <= bound, name
        assert (got.cpu()[z < -0.05] == 0).all(), f"{name}: a closed gate lets something through"
    ops.check_device_errors()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("neighbours", [False, True])
@pytest.mark.parametrize("nh,nkv,dk,dv,rot,D,page,norm", [(6, 3, 16, 24, 8, 32, 16, False), (5, 5, 20, 28, 12, 32, 8, False), (4, 2, 64, 48, 64, 64, 32, False),
                                                        (4, 1, 128, 128, 96, 128, 16, True), (2, 1, 48, 40, 0, 48, 4, False), (3, 1, 200, 64, 130, 208, 16, True),
                                                        (4, 1, 128, 128, 96, 128, 16, False), (2, 2, 256, 64, 128, 256, 16, False), (3, 3, 12, 12, 4, 16, 8, False)])
def test_rotation_then_unit_heads_then_the_paged_write(ops, dtype, neighbours, nh, nkv, dk, dv, rot, D, page, norm):
    T, n_pages, eps = 9, 7, 1e-3          # a large eps: where it stands matters
    pad = 3 if norm or dk == 20 else 4      # rows of four-entry vectors, and rows that are not
    W = nh * dk + nkv * (dk + dv) + pad
    proj = bf16_exact(T, W, scale=0.1, seed=dk)
    pos = torch.tensor([0, 1, 2, 3, 77, 78, 500, 511, 600])
    scaling = {"factor": 8.0, "original": 64, "fast": 4.0, "slow": 0.5} if neighbours else None
    cos, sin = tables(ops, pos, 300.0, rot, scaling) if rot else (None, None)
    gain = bf16_exact(dk, seed=5) + 1 if norm else None
    slots = torch.randperm(page * n_pages, generator=torch.Generator().manual_seed(dk))[:T]
    cache = torch.full((n_pages, 2, nkv, page, D), 7.0, dtype=dtype, device="cuda")
    gw = gain.float().cuda() if norm else None
    q = ops.qk_norm_rope_write(proj.to(dtype).cuda(), 0, nh * dk, nh * dk + nkv * dk, gw, gw, eps, cos, sin, cache, slots.int().cuda(), nh, nkv,
                               dk, dv, D, rot, page, neighbours=neighbours, post_norm=True)

    def turned(v):
        v = GP.unit_rms(v, eps) * gain if norm else v
        v = GP.rotate(v, pos, 300.0, rot, "neighbours" if neighbours else "half", scaling) if rot else v
        return GP.unit_rms(v, eps)
    want_q = turned(proj[:, :nh * dk].view(T, nh, dk))
    want_k = turned(proj[:, nh * dk:nh * dk + nkv * dk].view(T, nkv, dk))
    want_v = proj[:, nh * dk + nkv * dk:W - pad].view(T, nkv, dv)
    got = q.view(T, nh, D)
    close(got[..., :dk], want_q, dtype, "queries", atol32=2e-4)
    flat = cache.permute(0, 3, 1, 2, 4).reshape(-1, 2, nkv, D)[slots.cuda()]
    close(flat[:, 0, :, :dk], want_k, dtype, "keys", atol32=2e-4)
    close(flat[:, 1, :, :dv], want_v, dtype, "values")
    assert (got[..., dk:] == 0).all() and (flat[:, 0, :, dk:] == 0).all() and (flat[:, 1, :, dv:] == 0).all()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("halves", [False, True])
@pytest.mark.parametrize("nh,dq,rank,rope,rot,page,parts", [(3, 10, 24, 8, 8, 16, 0), (5, 20, 36, 12, 8, 8, 2), (8, 64, 192, 32, 32, 32, 0), (72, 16, 64, 16, 16, 4, 3),
                                                          (2, 8, 20, 0, 0, 8, 0)])
def test_latent_norm_rotations_and_paged_write_from_one_projection(ops, dtype, halves, nh, dq, rank, rope, rot, page, parts):
    """Queries, latent and key part from one projection row (a tensor, or a split product's partial sums): the latent's
    norm, the rotation of the key part and of every query's rotated part, in either pairing; a token whose slot is
    negative stores nothing but still gets its queries."""
    T, n_pages, col = 9, 6, 5
    c_col = col + nh * (dq + rope)
    W = c_col + rank + rope + 2
    row = -(-(rank + rope) // 16) * 16
    proj = bf16_exact(max(parts, 1), T, W, seed=rank)
    full = proj.sum(0)
    wc = bf16_exact(rank, seed=13) + 1
    pos = torch.tensor([0, 1, 2, 3, 77, 78, 500, 511, 600])
    slots = torch.randperm(page * n_pages, generator=torch.Generator().manual_seed(rank))[:T]
    slots[4] = -1
    cos, sin = tables(ops, pos, 1000.0, rot) if rot else (None, None)
    cache = torch.full((n_pages, 1, 1, page, row), 7.0, dtype=dtype, device="cuda")
    qa = torch.full((T, nh, row), 5.0, dtype=dtype, device="cuda")
    src = ops.PartialSums(proj.float().cuda(), dtype) if parts else full.to(dtype).cuda()
    ops.latent_prepare(src, 0, 0, c_col, rank, rope, rot, None, wc.float().cuda(), 1e-5, cos, sin, cache, slots.int().cuda(), page, dtype,
                       halves=halves, q_out=qa, qh_col=col, dq=dq)
    layout = "half" if halves else "neighbours"
    seen = full if parts else full.to(dtype).double()
    turn = lambda v: GP.rotate(v, pos, 1000.0, rot, layout) if rot else v
    want = torch.cat([GP.unit_rms(seen[:, c_col:c_col + rank], 1e-5) * wc, turn(seen[:, c_col + rank:c_col + rank + rope])], dim=1)
    want_q = turn(seen[:, col:c_col].view(T, nh, dq + rope)[..., dq:])
    flat = cache.view(-1, row)
    live = slots >= 0
    close(flat[slots[live].cuda(), :rank + rope], want[live], dtype, "cache rows", atol32=2e-4)
    assert (flat[slots[live].cuda(), rank + rope:] == 0).all()
    untouched = torch.ones(page * n_pages, dtype=torch.bool)
    untouched[slots[live]] = False
    assert (flat[untouched.cuda()] == 7.0).all(), "a row of no token was written"
    if rope:
        close(qa[..., rank:rank + rope], want_q, dtype, "rotated queries", atol32=2e-4)
    assert (qa[..., :rank] == 5.0).all() and (qa[..., rank + rope:] == 0).all()
    # the kernel for queries that come from a product of their own
    qa2 = torch.full((T, nh, row), 5.0, dtype=dtype, device="cuda")
    ops.latent_rotate_q(seen[:, col:c_col].to(dtype).cuda().contiguous(), qa2, cos, sin, nh, dq, rope, rot, rank, halves=halves)
    close(qa2[..., rank:rank + rope], want_q, dtype, "rotated queries alone", atol32=2e-4)
    ops.check_device_errors()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("mma", [False, True])
@pytest.mark.parametrize("T,Hn,K,N,extra,W", [(5, 3, 16, 24, 8, 96), (130, 4, 32, 48, 16, 208), (70, 5, 20, 36, 12, 177), (300, 3, 72, 200, 8, 248)])
def test_a_product_per_head_out_of_a_wider_row(ops, dtype, mma, T, Hn, K, N, extra, W, monkeypatch):
    """The heads lie inside a projection row (each ``K + extra`` wide, of which the first K count): no copy is made."""
    monkeypatch.setattr(ops, "USE_GROUPED_MMA", mma)
    proj, w = bf16_exact(T, W, seed=21), bf16_exact(Hn, N, K, seed=22)
    x = proj[:, :Hn * (K + extra)].reshape(T, Hn, K + extra)
    want = torch.einsum("thk,hnk->thn", x[..., :K], w)
    view = proj.to(dtype).cuda()[:, :Hn * (K + extra)].unflatten(1, (Hn, K + extra))
    close(ops.headwise_linear(view, w.to(dtype).cuda()), want, dtype, "view", atol32=2e-5, rel16=4e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,Hn,start", [(1, 96, True), (5, 92, False), (40, 256, True), (300, 320, False)])
def test_the_stream_fed_with_the_embedding_again(ops, dtype, T, Hn, start):
    """x = W [x; x0] three times in a row, branches pending before the second and third; in bfloat16 the products'
    operands are rounded, their results are not."""
    from pyre_b200.parts.base import PartSpec, load_part, make_part
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    part = make_part("stream", PartSpec("feed_again", {"width": Hn, "tensor_name": ""}), dt, "cuda")
    w = bf16_exact(Hn, 2 * Hn, scale=Hn ** -0.5, seed=1)
    load_part(part, {"loop.in": w.to(dt).cuda()}, "loop.in")
    x0 = bf16_exact(T, Hn, seed=2)
    ctx = type("Ctx", (), {"scratch": {}})()
    xd = x0.float().cuda()
    part.begin(ctx, xd)
    x = x0.clone()
    if not start:
        xd += 1.5
        x += 1.5
    ones = torch.ones(Hn, device="cuda")
    low = dt == torch.bfloat16
    for n in range(3):
        a, f = bf16_exact(T, Hn, seed=10 + n), bf16_exact(2, T, Hn, seed=20 + n)
        pending = None
        if n:
            pending = ops.ScaledSum([(a.to(dt).cuda(), ones), (ops.PartialSums(f.float().cuda(), dt), ones)], dt)
            x = x + a + f.sum(0)
        x = GP.feed_again(x, x0, w, low)
        before = xd
        xd, left = part.forward(ctx, xd, pending, at_start=start and n == 0)
        assert left is None and xd is before and xd.dtype == torch.float32
        close(xd, x, dt, f"pass {n}", atol32=3e-5, rel16=1.5e-2)
        if low and n == 0:         # the stream itself is not rounded to 16 bits
            assert not torch.equal(xd, xd.to(torch.bfloat16).float())
    assert torch.equal(x0, bf16_exact(T, Hn, seed=2))
    ops.check_device_errors()


# --------------------------------------------------------------------------- latent attention with sinks and gates
def latent_case(nh, rank, rope, page, seed, lens, starts):
    g = torch.Generator().manual_seed(seed)
    kd, row = rank + rope, -(-(rank + rope) // 16) * 16
    rows_of, qa, positions, seqs = [], [], [], []
    for b, (n, s0) in enumerate(zip(lens, starts)):
        total = s0 + n
        rows = (torch.randn(total, kd, generator=g) * 0.5).to(torch.bfloat16).double()
        q = torch.randn(n, nh, kd, generator=g).to(torch.bfloat16).double()
        for k, j in enumerate([0, total - 1, (total - 1) // page * page, (total - 1) // page * page - 1, total // 2]):
            if 0 <= j < total:      # keys far back, at a page's border and the newest stand out
                rows[j] = (q[-1, k % nh] * (1.5 + 0.2 * k)).to(torch.bfloat16).double()
        rows_of.append(rows)
        qa.append(q)
        positions += list(range(s0, total))
        seqs += [b] * n
    n_pages = sum(-(-r.shape[0] // page) for r in rows_of) + 3
    perm = torch.randperm(n_pages, generator=g).tolist()
    pool = torch.full((n_pages, 1, 1, page, row), float("nan"), dtype=F64)
    table = torch.full((len(rows_of), max(-(-r.shape[0] // page) for r in rows_of)), -1, dtype=torch.int32)
    for b, r in enumerate(rows_of):
        for lp in range(-(-r.shape[0] // page)):
            table[b, lp] = pg = perm.pop()
            piece = r[lp * page:(lp + 1) * page]
            pool[pg, 0, 0, :piece.shape[0]] = 0
            pool[pg, 0, 0, :piece.shape[0], :kd] = piece
    return rows_of, torch.cat(qa), positions, seqs, pool, table, kd, row


@pytest.mark.parametrize("kernel", ["exact32", "exact16", "mma"])
@pytest.mark.parametrize("nh,rank,rope,page", [(3, 24, 8, 16), (7, 112, 16, 16), (8, 192, 32, 32), (72, 64, 16, 8), (5, 36, 12, 8), (2, 272, 16, 16)])
def test_sinks_and_gates_in_every_latent_kernel(ops, kernel, nh, rank, rope, page):
    """A score per head that joins the denominator once (some vanish, some dominate: the output then nearly disappears),
    a sigmoid gate per head and token from a wider row, each alone and together, with the keys in one share or several."""
    dtype = torch.float32 if kernel == "exact32" else torch.bfloat16
    lens, starts = [1, 1, 37, 2, 90, 64], [0, 250, 0, 97, 40, 400]
    rows_of, qa, positions, seqs, pool, table, kd, row = latent_case(nh, rank, rope, page, nh * 1000 + rank, lens, starts)
    if kernel == "mma" and not ops.latent_mma_ok(dtype, row):
        pytest.skip("rows too wide for the tensor-core kernel")
    scale, T = 1.0 / math.sqrt(kd), qa.shape[0]
    sink = torch.tensor([[-30.0, 0.5, 3.0, 8.0, 25.0][h % 5] for h in range(nh)], dtype=F64)
    proj = bf16_exact(T, nh + 11, scale=2.0, seed=7)
    col = 4
    pos_d, seq_d = (torch.tensor(v, dtype=torch.int32, device="cuda") for v in (positions, seqs))
    cu = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32, device="cuda")
    qa_d = torch.zeros(T, nh, row, dtype=dtype, device="cuda")
    qa_d[..., :kd] = qa.to(dtype).cuda()
    n_tiles = sum(-(-n // (64 // min(nh, 64))) for n in lens)

    def plain(with_sink, with_gate):
        out = torch.zeros(T, nh, rank, dtype=F64)
        for t in range(T):
            rows = rows_of[seqs[t]][:positions[t] + 1]
            s = (qa[t] @ rows.T * scale).view(nh, 1, -1)
            p = GP.softmax_sink(s, torch.ones_like(s, dtype=torch.bool), sink if with_sink else None)
            out[t] = p[:, 0] @ rows[:, :rank]
            if with_gate:
                out[t] *= torch.sigmoid(proj[t, col:col + nh]).view(-1, 1)
        return out
    for with_sink, with_gate in ((True, False), (False, True), (True, True)):
        want = plain(with_sink, with_gate)
        kw = dict(sink=sink.float().cuda() if with_sink else None, gate=(proj.to(dtype).cuda(), col) if with_gate else None)
        what = f"sink {with_sink}, gate {with_gate}"
        if kernel != "mma":
            got = ops.latent_attention_exact(qa_d, pool.to(dtype).cuda(), table.cuda(), seq_d, pos_d, rank, rope, scale, None, **kw)
            close(got, want, dtype, what, atol32=2e-5, rel16=2e-2)
        else:
            for splits in (1, 3):
                got = ops.latent_attention_mma(qa_d, pool.to(dtype).cuda(), table.cuda(), cu, pos_d, n_tiles, rank, scale, None, n_splits=splits, **kw)
                close(got, want, dtype, f"{what}, {splits} shares", rel16=2.5e-2)
    assert (plain(True, False) - plain(False, False)).abs().max() > 0.5, "the sinks of this case would not show"
    ops.check_device_errors()


# --------------------------------------------------------------------------- a window beside kept first tokens
CASES = [(1, 300), (1, 2), (1, 0), (70, 130), (40, 0), (150, 0), (33, 61), (2, 411), (200, 300)]       # (new tokens, tokens cached before)


@pytest.mark.parametrize("kernel,dtype,nh,nkv,hd,page,window,keep", [
    ("generic", torch.float32, 6, 3, 48, 4, 37, 5), ("generic", torch.bfloat16, 3, 1, 32, 8, 19, 16), ("generic", torch.float32, 4, 2, 16, 16, 64, 33),
    ("generic", torch.float32, 2, 2, 144, 16, 1, 1), ("generic", torch.float32, 2, 1, 16, 8, 40, 100),
    ("mma", torch.bfloat16, 6, 3, 48, 4, 37, 5), ("mma", torch.bfloat16, 7, 1, 128, 8, 50, 20), ("mma", torch.bfloat16, 28, 4, 128, 16, 64, 16),
    ("mma", torch.bfloat16, 4, 1, 64, 32, 33, 17), ("mma", torch.bfloat16, 5, 5, 16, 12, 1, 1), ("mma", torch.bfloat16, 4, 2, 64, 16, 20, 130),
    ("mma", torch.bfloat16, 2, 1, 64, 8, 7, 3), ("mma", torch.bfloat16, 16, 1, 64, 64, 90, 70),
    ("prefill", torch.bfloat16, 6, 3, 128, 8, 50, 20), ("prefill", torch.bfloat16, 4, 2, 64, 12, 37, 65), ("prefill", torch.bfloat16, 2, 1, 64, 16, 5, 1),
    ("tc", torch.bfloat16, 6, 3, 128, 8, 50, 20), ("tc", torch.bfloat16, 4, 1, 64, 4, 37, 65), ("tc", torch.bfloat16, 28, 4, 128, 16, 64, 64),
    ("tc", torch.bfloat16, 4, 2, 64, 32, 136, 130), ("tc", torch.bfloat16, 2, 2, 128, 128, 1, 1)])
def test_kept_first_tokens_in_every_attention_kernel(ops, kernel, dtype, nh, nkv, hd, page, window, keep):
    """Entries that start everywhere (at position 0, inside the kept tokens, where the window still touches them, far
    behind), every token against the plain softmax over exactly its visible keys.  The last kept key, the first one
    that is not kept, and both edges of the last token's window stand out; pages that hold no visible key are absent,
    what a live page does not hold is NaN."""
    g = torch.Generator().manual_seed(nh * 7 + page + keep)
    cases = [c for c in CASES if c[0] >= {"prefill": 32, "tc": 64}.get(kernel, 0)]
    lens, starts = [n for n, _ in cases], [s for _, s in cases]
    scale = hd ** -0.5
    keys, values, queries, positions, seqs = [], [], [], [], []
    for b, (n, s0) in enumerate(cases):
        total = s0 + n
        k, v = torch.randn(total, nkv, hd, generator=g), torch.randn(total, nkv, hd, generator=g)
        q = torch.randn(n, nh, hd, generator=g)
        k, q = k.to(torch.bfloat16).double(), q.to(torch.bfloat16).double()
        last = total - 1
        for m, j in enumerate([keep - 1, keep, last - window + 1, last - window, 0]):
            if 0 <= j <= last:
                for gh in range(nkv):
                    k[j, gh] = (q[-1, gh * (nh // nkv)] * (1.0 + 0.15 * m)).to(torch.bfloat16).double()
        keys.append(k)
        values.append(v.to(torch.bfloat16).double())
        queries.append(q)
        positions += list(range(s0, total))
        seqs += [b] * n
    n_pages = sum(-(-len(k) // page) for k in keys) + 2
    perm = torch.randperm(n_pages, generator=g).tolist()
    pool = torch.full((n_pages, 2, nkv, page, hd), float("nan"), dtype=F64)
    width = max(-(-len(k) // page) for k in keys)
    table = torch.full((len(cases), width), -1, dtype=torch.int32)
    for b, (k, v) in enumerate(zip(keys, values)):
        first_window_page = max(0, starts[b] - window + 1) // page
        for lp in range(-(-len(k) // page)):
            if -(-keep // page) <= lp < first_window_page:
                continue
            table[b, lp] = pg = perm.pop()
            for name, src in ((0, k), (1, v)):
                piece = src[lp * page:(lp + 1) * page]
                pool[pg, name, :, :piece.shape[0]] = piece.transpose(0, 1)
    q = torch.cat(queries)
    want = torch.zeros(len(positions), nh, hd, dtype=F64)
    for b, (n, s0) in enumerate(cases):
        seen = GP.visible(s0 + n, window, keep)[s0:]
        kk, vv = (x.repeat_interleave(nh // nkv, dim=1) for x in (keys[b], values[b]))
        qb = q[[i for i, s in enumerate(seqs) if s == b]]
        p = GP.softmax_sink(torch.einsum("ihd,jhd->hij", qb, kk) * scale, seen)
        want[[i for i, s in enumerate(seqs) if s == b]] = torch.einsum("hij,jhd->ihd", p, vv)
    T = len(positions)
    qd = q.view(T, nh * hd).to(dtype).cuda()
    cache, tab = pool.to(dtype).cuda(), table.cuda()
    pos_d, seq_d = (torch.tensor(v, dtype=torch.int32, device="cuda") for v in (positions, seqs))
    cu = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32, device="cuda")
    runs = {}
    if kernel == "generic":
        runs["whole"] = ops.paged_attention_generic(qd, cache, tab, seq_d, pos_d, nh, nkv, hd, scale, window, keep_first=keep)
    elif kernel == "mma":
        for splits in (1, 3, 9, 24):      # whole, clusters, scratch and the combining kernel
            runs[f"{splits} splits"] = ops.paged_attention_mma(qd, cache, tab, cu, pos_d, len(cases), nh, nkv, hd, scale, window, splits, keep_first=keep)
    elif kernel == "prefill":
        runs["whole"] = ops.attention_prefill(qd, cache, tab, cu, pos_d, len(cases), T, nh, nkv, hd, scale, window, torch.zeros_like(qd), min_len=32, keep_first=keep)
    else:
        for shares in (1, 3):
            runs[f"{shares} shares"] = ops.attention_prefill_tc(qd, cache, tab, cu, pos_d, len(cases), T, nh, nkv, hd, scale, window, torch.zeros_like(qd),
                                                                min_len=64, key_splits=shares, keep_first=keep)
    ops.check_device_errors()
    for what, got in runs.items():
        assert torch.isfinite(got).all(), f"{what}: non-finite outputs"
        close(got.view(T, nh, hd), want, dtype, what, atol32=2e-5, rel16=2.5e-2)


# --------------------------------------------------------------------------- each mixer alone, through the cache manager
def run_mixer_alone(tmp_path, layer, width, eps, dtype, page, steps, inputs, seed):
    """The one mixer of a one-layer model on inputs of the test's own, on the step contexts that the package's stepper
    builds for ``steps`` (lists of (request, tokens) per step; a request begins at its first entry and ends after its
    last).  Returns the mixer's rows per request and the weights."""
    from pyre_b200.engine.replay import runtime_for_model
    from pyre_b200.engine.step import StepEntry
    from pyre_b200.kernels import ops
    from pyre_b200.models.model import load_model
    from safetensors.torch import load_file
    raw = {"architecture": "Gadopel", "vocab": 32, "width": width, "norm": {"eps": eps}, "layers": [dict(layer, mlp=None)]}
    GH.make_gadopel_dir(tmp_path, raw, seed=seed)
    model, _ = load_model(tmp_path, "cuda", dtype)
    last = {r: i for i, st in enumerate(steps) for r, _ in st}
    as_trace = [{"entries": [{"id": r, "tokens": [0] * n} for r, n in st], "end": [r for r, _ in st if last[r] == i]} for i, st in enumerate(steps)]
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
        for r, _ in step:
            if last[r] == i:
                cache.end(r)
    ops.check_device_errors()
    cache.check()
    assert not cache.live()
    return {r: torch.cat(v) for r, v in out.items()}, load_file(str(tmp_path / "model.safetensors"))


LENGTHS_ALONE = {"a": 1, "b": 2, "c": 50, "d": 33, "e": 150, "f": 17, "g": 90}


def mixer_schedule(seed):
    """Steps of up to three live requests, portions of 1 to 80 tokens; seven requests in all, so pages are used again."""
    rng = np.random.default_rng(seed)
    waiting, live, left, steps = list(LENGTHS_ALONE.items()), [], {}, []
    while waiting or live:
        while waiting and len(live) < 3:
            r, n = waiting.pop(0)
            live.append(r)
            left[r] = n
        step = []
        for r in list(live):
            n = min(left[r], int(rng.choice([1, 1, 2, 5, 9, 30, 80])))
            step.append((r, n))
            left[r] -= n
            if not left[r]:
                live.remove(r)
        steps.append(step)
    return steps


def check_mixer(tmp_path, layer, width, dtype, page, plain, seed, wrong=()):
    inputs = {r: bf16_exact(n, width, seed=seed + i) for i, (r, n) in enumerate(LENGTHS_ALONE.items())}
    got, w = run_mixer_alone(tmp_path, layer, width, 1e-5, dtype, page, mixer_schedule(seed), inputs, seed)
    for r, h in inputs.items():
        want = plain(h, w)
        size = float(want.abs().max())
        err = (got[r].double() - want).abs()
        bad = (err > (2e-5 if dtype == "float32" else 3e-2) * (size + want.abs())).any(dim=1)
        assert not bad.any(), f"request {r}: first wrong token {int(torch.where(bad)[0][0])} of {h.shape[0]}, max error {float(err.max()):.3e} of {size:.3e}"
    # the test can see the faults it is there for: the plain result with one is far outside the bound
    h = inputs["e"]
    want = plain(h, w)
    for other in wrong:
        assert ((other(h, w) - want).abs() > 2 * 3e-2 * (float(want.abs().max()) + want.abs())).any(), "this case would not show the fault"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv,dk,dv,window,keep,rot,page,width", [
    (6, 3, 16, 24, 11, 3, 8, 16, 96), (5, 5, 20, 28, 7, 1, 12, 8, 92), (4, 2, 64, 48, 64, 20, 64, 32, 256), (6, 1, 48, 40, 100000, 5, 16, 16, 128),
    (2, 2, 32, 32, 1, 1, 16, 16, 64), (2, 1, 16, 16, 16, 16, 16, 16, 64), (3, 1, 32, 16, 17, 33, 32, 16, 72), (4, 1, 128, 128, 40, 70, 96, 16, 128),
    (2, 1, 64, 128, 90, 2, 32, 64, 128), (3, 3, 12, 12, 9, 0, 12, 8, 92)])
def test_windowed_attention_with_kept_tokens_alone(tmp_path, dtype, heads, kv, dk, dv, window, keep, rot, page, width):
    layer = GH.attn(heads, kv, dk, dv, 3.0 / math.sqrt(dk), window, keep, rot, 100.0, (8.0, 32, 4.0, 1.0))
    mx = layer["mixer"]

    def plain(h, w, m=mx):
        return GP.attention(h, w, "l0.mix.", m, 1e-5)
    wrong = []
    if window < 140:
        for dw, dk_ in ((1, 0), (-1, 0), (0, 1), (0, -1)):
            if window + dw > 0 and keep + dk_ >= 0:
                wrong.append(lambda h, w, dw=dw, dk_=dk_: plain(h, w, dict(mx, mask={"size": window + dw, "keep_first": keep + dk_})))
    check_mixer(tmp_path, layer, width, dtype, page, plain, seed=heads + window, wrong=wrong if dtype == "float32" and window + keep < 60 else ())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,rot,dv,rank,page,width", [(3, 16, 8, 24, 40, 16, 96), (5, 20, 12, 12, 36, 8, 92), (8, 64, 32, 64, 192, 32, 256),
                                                             (72, 16, 16, 8, 64, 16, 128), (1, 24, 4, 40, 20, 16, 64), (2, 32, 2, 16, 300, 16, 72)])
def test_latent_attention_alone(tmp_path, dtype, heads, dim, rot, dv, rank, page, width):
    layer = GH.latent(heads, dim, rot, dv, rank, 1.0 / math.sqrt(dim + rot), 300.0)
    mx = layer["mixer"]

    def plain(h, w):
        return GP.latent_attention(h, w, "l0.mix.", mx, 1e-5)
    wrong = [lambda h, w: plain(h, dict(w, **{"l0.mix.sink": w["l0.mix.sink"] - 60.0})),        # no sink
             lambda h, w: plain(h, dict(w, **{"l0.mix.g": w["l0.mix.g"] * 0}))]                 # every gate one half
    check_mixer(tmp_path, layer, width, dtype, page, plain, seed=heads, wrong=wrong)


# --------------------------------------------------------------------------- the engine against the plain model
LENGTHS = {"A": [1, 2, 17, 33, 70, 130], "B": [5, 31, 97, 120], "C": [3, 63, 64, 65, 260], "D": [2, 47, 129]}
LONG = {"A": [220, 190], "C": [250, 180]}      # decoded one by one from token 70 (40) on


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for n, (name, raw) in enumerate(GH.GAD.items()):
        d = tmp_path_factory.mktemp(f"gadopel_{name}")
        GH.make_gadopel_dir(d, raw, seed=700 + n)
        reqs = {f"{name}{i}": GH.random_ids(raw, L, seed=13 * n + i) for i, L in enumerate(LENGTHS[name])}
        plain = {rid: GH.plain_logits(d, ids) for rid, ids in reqs.items()}
        lowp = {rid: GH.plain_logits(d, ids, lowp=True) for rid, ids in reqs.items()}
        sq = sum(float(((lowp[rid] - plain[rid]) ** 2).sum()) for rid in reqs)
        long_reqs = {f"long{i}": GH.random_ids(raw, L, seed=90 + i) for i, L in enumerate(LONG.get(name, []))}
        long_plain = {r: (GH.plain_logits(d, ids), GH.plain_logits(d, ids, lowp=True)) for r, ids in long_reqs.items()}
        out[name] = (d, reqs, plain, math.sqrt(sq / sum(p.size for p in plain.values())), lowp, long_reqs, long_plain)
    return out


def run(models, name, dtype, steps, what, rename=None):
    d, reqs, plain, lowp_rms, lowp = models[name][:5]
    got = H.run_trace_in_process(d, dtype, steps, H.max_live_tokens(steps), GH.GAD_PAGE_SIZE[name])
    if rename:
        plain, lowp = ({new: src[old] for new, old in rename.items()} for src in (plain, lowp))
    GH.compare(got, plain, dtype, what, lowp_rms, lowp)


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_the_stream_after_every_layer_run(models, name):
    """In 32-bit, the stream after each layer run against the plain implementation's: the first that differs is named."""
    from pyre_b200.engine.replay import runtime_for_model
    from pyre_b200.engine.step import StepEntry
    from pyre_b200.kernels import ops
    from pyre_b200.models.model import load_model
    from safetensors.torch import load_file
    d, reqs = models[name][:2]
    ids = max(reqs.values(), key=len)[:60]
    want = []
    with torch.inference_mode():
        GP.forward(ids, load_file(str(d / "model.safetensors")), GH.GAD[name], streams=want)
    model, _ = load_model(d, "cuda", "float32")
    got = []

    def recorded(forward):
        def run_layer(ctx, x, pending, call):
            x, pending = forward(ctx, x, pending, call)
            got.append((x + ops.materialize(pending).float() if pending is not None else x).double().cpu())
            return x, pending
        return run_layer
    for b in model.blocks:
        b.forward = recorded(b.forward)
    cache, stepper = runtime_for_model(model, 64, GH.GAD_PAGE_SIZE[name], max_requests=1, cuda_graphs=False)
    cache.begin("r")
    stepper.step([StepEntry("r", ids, [])])
    assert len(got) == len(want) == len(model.calls)
    for n, (g, w) in enumerate(zip(got, want)):
        err = (g - w).abs().max()
        assert err < 2e-4 * (1 + w.abs().max()), f"layer run {n} (layer {model.calls[n].block}): off by {float(err):.3e}"
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
def test_mixed_batches_reuse_pages(models, name, dtype):
    """Every request twice under other names, at most four alive: later ones get the pages (filled with NaN when
    they were given back, by a window or at the end) that earlier ones held, and must come out as each alone."""
    reqs = models[name][1]
    many = {f"{rid}r{rep}": ids for rep in range(2) for rid, ids in reqs.items()}
    steps = H.trace_mixed(many, seed=21, max_live=4, portion=(2, 40))
    run(models, name, dtype, steps, "mixed", rename={f"{rid}r{rep}": rid for rep in range(2) for rid in reqs})


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_cutting_and_batching_change_no_bit_in_32_bit(models, name):
    d, reqs = models[name][:2]
    page = GH.GAD_PAGE_SIZE[name]
    whole = H.run_trace_in_process(d, "float32", H.trace_whole(reqs), 2048, page)
    mixed_steps = H.trace_mixed(reqs, seed=3, max_live=4, portion=(2, 40))
    mixed = H.run_trace_in_process(d, "float32", mixed_steps, H.max_live_tokens(mixed_steps), page)
    for rid in reqs:
        assert np.array_equal(whole[rid], mixed[rid]), f"{rid}: max {np.abs(whole[rid] - mixed[rid]).max():.3e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding(models, name, dtype):
    """Up to 250 tokens, most of them one by one (captured decode steps), two requests side by side: every window passes
    over decoded tokens several times and gives pages back on the way; the kept first tokens stay."""
    d, lowp_rms, reqs, long_plain = models[name][0], models[name][3], models[name][5], models[name][6]
    steps = [{"step": 0, "entries": [{"id": r, "tokens": ids[:70 - 30 * i], "want": [0]} for i, (r, ids) in enumerate(reqs.items())], "end": []}]
    at = {r: 70 - 30 * i for i, r in enumerate(reqs)}
    while any(at[r] < len(reqs[r]) for r in reqs):
        entries = [{"id": r, "tokens": [reqs[r][at[r]]], "want": [0]} for r in reqs if at[r] < len(reqs[r])]
        for e in entries:
            at[e["id"]] += 1
        steps.append({"step": len(steps), "entries": entries, "end": [e["id"] for e in entries if at[e["id"]] == len(reqs[e["id"]])]})
    got = H.run_trace_in_process(d, dtype, steps, H.max_live_tokens(steps), GH.GAD_PAGE_SIZE[name])
    want, lowp = {}, {}
    for i, r in enumerate(reqs):
        for dst, full in ((want, long_plain[r][0]), (lowp, long_plain[r][1])):
            dst[r] = np.concatenate([full[:1], full[70 - 30 * i:]])
    GH.compare(got, want, dtype, "long decoding", lowp_rms, lowp)


@pytest.mark.parametrize("name,seqs,pages", [("A", 3, 5), ("C", 3, 5), ("B", 3, 12), ("A", 6, 14)])
def test_greedy_generation_through_the_engine(models, name, seqs, pages):
    """``Engine.generate`` (scheduler, portions of prompts, captured decode steps, sampler) gives the tokens that
    the plain implementation's argmax gives, in 32-bit; a cache too small for all requests at once makes the
    scheduler preempt and recompute; six requests side by side decode in captured steps that are padded with rows of no
    request."""
    from pyre_b200.engine.engine import Engine
    from pyre_b200.sampling import SamplingParams
    d = models[name][0]
    raw = GH.GAD[name]
    prompts = [H.random_ids(raw["vocab"], n, seed=40 + n) for n in ((15, 16, 3, 30) if seqs == 3 else (15, 16, 3, 30, 7, 11))]
    new = 12
    engine = Engine(str(d), dtype="float32", page_size=16, num_pages=pages, max_num_seqs=seqs, max_num_batched_tokens=32, prefill_chunk=20)
    outs = engine.generate(prompts, SamplingParams(max_new_tokens=new, return_logits=True))
    for p, o in zip(prompts, outs):
        ids = list(p)
        for k in range(new):
            logits = GH.plain_logits(d, ids)[-1]
            top2 = np.sort(logits)[-2:]
            np.testing.assert_allclose(o.logits[k], logits, rtol=2e-4, atol=1e-4)
            if top2[1] - top2[0] > 2e-4:
                assert o.token_ids[k] == int(logits.argmax()), f"token {k} of a prompt of {len(p)}"
            ids.append(o.token_ids[k])
    assert json.dumps(engine.stats())
