"""Gugidra on the host side: the configuration, the registry, the model as data, and (with plain torch stand-ins for the
kernels) the package's own parts, cache manager, step function and replay loop against the plain implementation, under
cutting, batching and reuse of pages and state slots."""

import json

import numpy as np
import pytest
import torch

import gugidra_helpers as GH
import helpers as H
import standins
from plain import gugidra_plain as GP
from pyre_b200.config import ConfigError, config_from_dict, load_config
from pyre_b200.config.model_config import GugidraConfig
from pyre_b200.config.registry import architecture_of
from pyre_b200.models.model import Model, tensor_table


def test_config_round_trip_and_registry():
    for raw in GH.GUG.values():
        cfg = config_from_dict(raw)
        assert isinstance(cfg, GugidraConfig)
        assert config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    a = config_from_dict(GH.GUG_A)
    assert [L.kind for L in a.layers] == ["parallel", "gla", "parallel", "gla"] and [L.mlp_kind for L in a.layers] == ["dense", "moe", "", "dense"]
    assert (a.embedding_scale, a.logit_softcap, a.loop_start, a.loop_stop, a.loop_times) == (3.0, 1.5, 1, 3, 3)
    L = a.layers[1]
    assert (L.experts, L.top, L.group_count, L.group_keep, L.ff, L.limit, L.shared_ff, L.shared_limit, L.tau) == (6, 2, 3, 2, 32, 0.6, 40, 1.1, 8.0)
    assert a.layer_order() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    b = config_from_dict(GH.GUG_B)
    assert (b.embedding_scale, b.logit_softcap, b.has_loop(), b.layers[0].group_count, b.layers[0].shared_ff) == (1.0, 0.0, False, 1, 0)


@pytest.mark.parametrize("edit, word", [
    (lambda r: r["layers"][1].update(type="conv"), "type"),
    (lambda r: r["layers"][1]["mixer"].pop("tau"), "tau"),
    (lambda r: r["layers"][0]["mixer"].pop("right"), "right"),
    (lambda r: r["layers"][0]["mixer"]["right"].pop("gate_cap"), "gate_cap"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=34), "rot"),
    (lambda r: r["layers"][0]["mixer"]["left"].update(vdim=16), "vdim"),
    (lambda r: r["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda r: r["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=5), "top"),
    (lambda r: r["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda r: r["layers"][1]["mlp"]["shared"].pop("limit"), "limit"),
    (lambda r: r["loop"].update(stop=5), "loop"),
    (lambda r: r.pop("norm"), "norm"),
])
def test_config_errors_name_the_key(edit, word):
    raw = json.loads(json.dumps(GH.GUG_A))
    edit(raw)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(raw)


def test_tensor_names_cache_groups_and_state_groups():
    cfg = config_from_dict(GH.GUG_A)
    spec = architecture_of(cfg).build(cfg)
    table = tensor_table(spec)
    assert {"embed", "head", "final.norm", "loop.step", "l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.mix.left.q", "l0.mix.left.q.b",
            "l0.mix.left.k", "l0.mix.left.k.b", "l0.mix.left.o", "l0.mix.left.o.b", "l0.mix.right.q", "l0.mix.right.i", "l0.mix.right.i.b",
            "l0.mix.right.f", "l0.mix.right.f.b", "l0.mix.right.norm", "l0.mix.right.g", "l0.mix.right.o", "l0.mlp.gate", "l0.mlp.up", "l0.mlp.down",
            "l1.mix.q", "l1.mix.a1", "l1.mix.a2", "l1.mix.a2.b", "l1.mix.norm", "l1.mix.g", "l1.mlp.router", "l1.mlp.correction", "l1.mlp.e5.down",
            "l1.mlp.shared.gate"} <= set(table)
    assert not {"l0.mix.left.v", "l0.mix.left.v.b", "l2.mlp.router", "l1.mlp.e6.up", "l0.mix.right.q.b"} & set(table)
    assert table["l2.norm2"].optional and table["l2.norm2b"].optional and not table["l0.norm2"].optional
    assert table["loop.step"].shape == (3, 96) and table["l1.mix.norm"].shape == (24,) and table["l0.mix.right.norm"].shape == (72,)
    assert table["l0.mix.left.k"].shape == (64, 96) and table["l1.mix.a2"].shape == (48, 6) and table["l1.mix.a1"].shape == (6, 96)
    model = Model(spec, torch.float32, "cpu")
    # every pass of the repeated span has a cache layer and state of its own
    assert sorted((g.spec.n_kv_heads, g.spec.head_dim, g.n_layers) for g in model.kv_groups) == [(1, 16, 3), (2, 32, 1)]
    mem = lambda H, d, v: (H * (d * v + d + -(-v // 16) + 1),)
    assert sorted((g.spec.shape, g.n_layers) for g in model.state_groups) == sorted([(mem(3, 16, 24), 1), ((3 * 16 * 24,), 3), (mem(2, 24, 40), 3), ((2 * 40 * 16,), 1)])
    assert {"matrix_state", "grouped", "blockops", "attention_generic", "parallel_block"} <= set(model.kernel_libraries())
    assert [(c.add_embedding, c.add_vector and c.add_vector[1]) for c in model.calls] == \
        [(False, None), (False, 0), (False, None), (True, 1), (False, None), (True, 2), (False, None), (False, None)]


def test_a_size_that_the_file_leaves_out_comes_from_the_tensor(tmp_path):
    GH.make_gugidra_dir(tmp_path, GH.GUG_B, seed=1)
    raw = json.loads(json.dumps(GH.GUG_B))
    raw["layers"][0]["mixer"].pop("decay_rank")
    raw["layers"][2]["mixer"].pop("decay_rank")
    (tmp_path / "config.json").write_text(json.dumps(raw))
    assert config_from_dict(raw).needs_tensor_shapes()
    cfg = load_config(tmp_path)
    assert (cfg.layers[0].decay_rank, cfg.layers[2].decay_rank) == (5, 9) and cfg == config_from_dict(GH.GUG_B)


def test_side_by_side_takes_stacked_mixers_with_one_cache_and_one_state():
    from pyre_b200.kernels.ops import UnsupportedSize
    from pyre_b200.parts.base import PartSpec, make_part
    memory = PartSpec("matrix_memory", {"width": 32, "n_heads": 1, "head_dim": 8, "v_head_dim": 8, "gate_cap": 5.0, "eps": 1e-5})
    with pytest.raises(UnsupportedSize, match="state"):
        make_part("mixer", PartSpec("side_by_side", {"branches": (("a.", memory, 1.0), ("b.", memory, 1.0))}), torch.float32, "cpu")
    wkv = PartSpec("wkv", {"width": 32, "n_heads": 1, "head_dim": 8, "decay_rank": 4, "eps": 1e-5})
    with pytest.raises(ValueError, match="StackedMixer"):
        make_part("mixer", PartSpec("side_by_side", {"branches": (("a.", memory, 1.0), ("b.", wkv, 1.0))}), torch.float32, "cpu")


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for n, name in enumerate(["A", "B", "D"]):
        d = tmp_path_factory.mktemp(f"gug_{name}")
        GH.make_gugidra_dir(d, GH.GUG[name], seed=300 + n)
        reqs = {f"{name}{i}": GH.decided_ids(d, L, seed=17 * n + i) for i, L in enumerate([1, 2, 19, 37, 50])}
        out[name] = (d, reqs, {rid: GH.plain_logits(d, ids) for rid, ids in reqs.items()})
    return out


def _replay_on_cpu(monkeypatch, folder, steps, page_size, max_requests=4):
    import tempfile
    from pathlib import Path
    from pyre_b200.engine import replay as rp
    from pyre_b200.models.model import load_model

    standins.install(monkeypatch)
    model, _cfg = load_model(folder, "cpu", "float32")
    cache, stepper = rp.runtime_for_model(model, H.max_live_tokens(steps), page_size, max_requests, poison=True, cuda_graphs=False)
    with tempfile.TemporaryDirectory() as out:
        rp.replay(stepper, [json.dumps(s) for s in steps], Path(out), done=lambda m: None)
        got = H.collect_trace_logits(steps, lambda n: np.fromfile(Path(out) / f"{n}.f32", dtype="<f4").reshape(-1, model.vocab_size))
    cache.check()
    assert not cache.live() and cache.state.num_free == max_requests
    return got


@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_host_side_portions_and_mixed_batches(monkeypatch, folders, name):
    d, reqs, plain = folders[name]
    steps = []
    for k, (rid, ids) in enumerate(reqs.items()):
        steps += H.trace_portions(rid, ids, [[2, 9, 3], [5, 2, 16]][k % 2], first_step=len(steps))
    GH.compare(_replay_on_cpu(monkeypatch, d, steps, GH.GUG_PAGE_SIZE[name]), plain, "float32", "portions")
    many = {f"{rid}r{rep}": ids for rep in range(2) for rid, ids in reqs.items()}     # ten requests, four alive at a time:
    steps = H.trace_mixed(many, seed=5, max_live=4)                                   # pages and state slots are used again
    got = _replay_on_cpu(monkeypatch, d, steps, GH.GUG_PAGE_SIZE[name])
    GH.compare(got, {f"{rid}r{rep}": plain[rid] for rep in range(2) for rid in reqs}, "float32", "mixed")


@pytest.mark.parametrize("fault", ["correction", "groups", "group of masked zeros", "keep", "limit", "up", "tau", "cap",
                                   "rotated values", "bias", "scales", "pass vector", "embedding again", "softcap"])
def test_the_models_would_show_a_fault(monkeypatch, folders, fault):
    """Each mechanism misread on purpose in the plain implementation moves the logits of one of the test models far beyond
    what the comparisons allow: the weights are such that it shows.  (The matrix memory's denominator is not among them: the
    unit norm per head takes a common factor off again, so it is compared where the kernel leaves it.)"""
    from safetensors.torch import load_file

    def gap(edit=None, weights=None):
        worst = 0.0
        for name, (d, reqs, plain) in folders.items():
            raw = json.loads(json.dumps(GH.GUG[name]))
            if edit:
                edit(raw)
            w = load_file(str(d / "model.safetensors"))
            if weights:
                weights(w)
            ids = reqs[f"{name}4"]
            with torch.inference_mode():
                worst = max(worst, float(np.abs(GP.forward(raw, w, ids).numpy() - plain[f"{name}4"]).max()))
        return worst

    def layers(fn):
        return lambda raw: [fn(L) for L in raw["layers"]]

    def zero(suffix):
        return lambda w: w.update({n: torch.zeros_like(t) for n, t in w.items() if n.endswith(suffix)})

    edit = weights = None
    if fault == "correction":
        weights = zero(".mlp.correction")
    elif fault == "groups":
        edit = layers(lambda L: ((L["mlp"] or {}).get("router") or {}).pop("groups", None))
    elif fault == "keep":
        edit = layers(lambda L: (((L["mlp"] or {}).get("router") or {}).get("groups") or {}).update(keep=1))
    elif fault == "group of masked zeros":
        # the experts of the groups left out compete with 0 instead of not at all
        def choose(scores, correction, router):
            choice, n = scores + correction, (router.get("groups") or {"count": 1})["count"]
            if n > 1:
                two = choice.view(-1, n, choice.shape[-1] // n).sort(-1, descending=True).values[..., :2].sum(-1)
                keep = torch.zeros_like(two, dtype=torch.bool).scatter(-1, two.topk(router["groups"]["keep"], -1).indices, True)
                choice = choice.masked_fill(~keep.repeat_interleave(choice.shape[-1] // n, -1), 0.0)
            return choice.topk(router["top"], -1).indices, []
        s = torch.tensor([[0.3, 0.2, 0.1, 0.05]])
        c = torch.tensor([-0.9, -0.9, -0.9, -0.9])
        router = {"top": 1, "groups": {"count": 2, "keep": 1}}
        assert int(choose(s, c, router)[0]) != int(GP.choose(s, c, router)[0]) == 0
        return
    elif fault == "limit":
        edit = layers(lambda L: L["mlp"] and (L["mlp"].update(limit=1e9) if L["mlp"]["kind"] == "dense" else L["mlp"]["expert"].update(limit=1e9)))
    elif fault == "up":
        monkeypatch.setattr(GP, "clamped_gate", lambda g, u, limit: torch.clamp(g, max=limit) * torch.sigmoid(1.702 * torch.clamp(g, max=limit)) * torch.clamp(u, -limit, limit))
    elif fault == "tau":
        edit = layers(lambda L: L["type"] == "gla" and L["mixer"].update(tau=L["mixer"]["tau"] * 1.5))
    elif fault == "cap":
        edit = layers(lambda L: L["type"] == "parallel" and L["mixer"]["right"].update(gate_cap=1e6))
    elif fault == "rotated values":
        def attention(h, w, prefix, m, lowp=False):
            T, H, d, G = h.shape[0], m["heads"], m["dim"], m["kv_heads"]
            g = lambda n: w[prefix + n].double()
            q, k = (h @ g("q").T + g("q.b")).view(T, H, d), (h @ g("k").T + g("k.b")).view(T, G, d)
            q, k = (GP.turn_neighbours(t, m["rot"]["base"], m["rot"]["dims"]) for t in (q, k))
            seen = torch.tril(torch.ones(T, T, dtype=torch.bool))
            out = torch.stack([torch.softmax(((q[:, n] @ k[:, n // (H // G)].T) * m["scale"]).masked_fill(~seen, -1e30), -1) @ k[:, n // (H // G)] for n in range(H)], 1)
            return out.reshape(T, H * d) @ g("o").T + g("o.b")
        monkeypatch.setattr(GP, "key_value_attention", attention)
    elif fault == "bias":
        weights = zero(("left.q.b", "left.k.b", "left.o.b"))
    elif fault == "scales":
        edit = layers(lambda L: L["type"] == "parallel" and L["mixer"].update(left_scale=1.0, right_scale=1.0))
    elif fault == "pass vector":
        weights = zero("loop.step")
    elif fault == "embedding again":
        real_order = GP.layer_order
        # every pass as if it were the first: the vector of its row is not what is at stake here
        monkeypatch.setattr(GP, "layer_order", lambda c: [(i, 0 if t is not None else None) for i, t in real_order(c)])
    elif fault == "softcap":
        edit = lambda raw: raw.pop("logit_softcap", None)
    assert gap(edit, weights) > 5e-2, f"{fault}: the test models would not show it"


def test_random_model_folder_loads(tmp_path, monkeypatch):
    from pyre_b200.models.model import load_model
    from pyre_b200.weights import write_random_model

    standins.install(monkeypatch)
    cfg = config_from_dict(GH.GUG_D)
    write_random_model(tmp_path, cfg, seed=1)
    assert json.loads((tmp_path / "config.json").read_text())["architecture"] == "Gugidra"
    model, loaded = load_model(tmp_path, "cpu", "float32")
    assert loaded == cfg and model.loaded
