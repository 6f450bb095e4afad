"""Gadopel on the host side: the configuration, the registry, the model as data, the cache manager's windows beside kept
first tokens, and (with plain torch stand-ins for the kernels) the package's own parts, cache manager, step function and
replay loop against the plain implementation, under cutting, batching and reuse of pages."""

import json

import numpy as np
import pytest
import torch

import gadopel_helpers as GH
import helpers as H
import standins
from plain import gadopel_plain as GP
from pyre_b200.config import ConfigError, config_from_dict
from pyre_b200.config.model_config import GadopelConfig
from pyre_b200.config.registry import architecture_of
from pyre_b200.models.model import KVGroup, Model, tensor_table
from pyre_b200.parts.base import PagedKVSpec


def test_config_round_trip_and_registry():
    for raw in GH.GAD.values():
        cfg = config_from_dict(raw)
        assert isinstance(cfg, GadopelConfig)
        assert config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    cfg = config_from_dict(GH.GAD_A)
    assert [L.kind for L in cfg.layers] == ["attention", "latent_attention", "attention", "latent_attention"]
    assert [(L.window, L.keep_first, L.ff) for L in cfg.layers] == [(11, 3, 160), (0, 0, 96), (29, 18, 0), (0, 0, 0)]
    assert cfg.layers[0].rot_scaling == (8.0, 32.0, 4.0, 1.0) and cfg.layers[0].kv_heads == 3 and cfg.layers[1].kv_rank == 40
    assert cfg.layer_order() == [(0, False), (1, True), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert cfg.layer_order() == GP.layer_order(GH.GAD_A)
    b = config_from_dict(GH.GAD_B)
    assert not b.has_loop() and b.layer_order() == [(i, False) for i in range(4)] and b.layers[1].rot_scaling is None
    raw = json.loads(json.dumps(GH.GAD_B))
    del raw["layers"][1]["mixer"]["mask"], raw["layers"][1]["mixer"]["rot"]      # neither window nor rotation
    plain = config_from_dict(raw)
    assert (plain.layers[1].window, plain.layers[1].rot_dims) == (0, 0) and config_from_dict(plain.to_dict()) == plain


@pytest.mark.parametrize("edit, word", [
    (lambda r: r["layers"][1].update(type="mamba2"), "type"),
    (lambda r: r["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda r: r["layers"][1]["mixer"].pop("rot_dim"), "rot_dim"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=18), "rot"),
    (lambda r: r["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda r: r["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda r: r["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda r: r["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda r: r["loop"].update(stop=5), "loop"),
    (lambda r: r["loop"].update(times=0), "times"),
    (lambda r: r.pop("norm"), "norm"),
])
def test_config_errors_name_the_key(edit, word):
    raw = json.loads(json.dumps(GH.GAD_A))
    edit(raw)
    with pytest.raises(ConfigError, match=word):
        config_from_dict(raw)


def test_tensor_names_and_cache_groups():
    cfg = config_from_dict(GH.GAD_A)
    spec = architecture_of(cfg).build(cfg)
    table = tensor_table(spec)
    assert {"embed", "head", "loop.in", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.q", "l0.mix.v", "l0.mlp.gate", "l1.mix.dkv.norm",
            "l1.mix.sink", "l1.mix.g", "l1.mix.uk", "l1.mix.uv", "l1.mix.o", "l2.mix.k", "l3.norm1"} <= set(table)
    assert table["l2.norm2"].optional and table["l3.norm2"].optional and not table["l0.norm2"].optional      # layers without a feed-forward
    assert not {"l2.mlp.up", "l0.mix.sink", "l0.mix.g", "l1.mix.k", "l1.mix.dq", "l0.mix.q_norm"} & set(table)
    assert table["loop.in"].shape == (96, 192) and table["l1.mix.q"].shape == (3 * 24, 96) and table["l1.mix.dkv"].shape == (48, 96)
    assert table["l1.mix.sink"].shape == (3,) and table["l1.mix.g"].shape == (3, 96) and table["l1.mix.uv"].shape == (72, 40)
    assert table["l0.mix.k"].shape == (48, 96) and table["l0.mix.v"].shape == (72, 96) and table["l0.mix.o"].shape == (96, 144)
    model = Model(spec, torch.float32, "cpu")
    # every pass of a repeated layer has a cache layer of its own; windows and kept tokens make groups
    groups = sorted((g.spec.planes, g.spec.n_kv_heads, g.spec.window or 0, g.spec.keep_first, g.n_layers) for g in model.kv_groups)
    assert groups == [(1, 1, 0, 0, 1), (1, 1, 0, 0, 3), (2, 2, 29, 18, 3), (2, 3, 11, 3, 1)]
    assert [c.before for c in model.calls] == [None, "loop.in", None, "loop.in", None, "loop.in", None, None]
    assert {"latent_attention", "parallel_block", "blockops", "seqmix", "attention_generic"} <= set(model.kernel_libraries())
    b = config_from_dict(GH.GAD_B)
    assert "loop.in" not in tensor_table(architecture_of(b).build(b))
    with pytest.raises(ValueError, match="none of the model's streams"):
        spec.schedule[0] = type(spec.schedule[0])(0, before="elsewhere")
        spec.__post_init__()


# --------------------------------------------------------------------------- windows beside kept first tokens
@pytest.mark.parametrize("page, window, keep", [(4, 6, 1), (4, 6, 4), (4, 6, 5), (4, 9, 9), (8, 3, 20), (16, 40, 7), (4, 1, 2)])
def test_the_kept_first_pages_stay(page, window, keep):
    """Every position that a later token may read is on a live page, the pages between the kept tokens and the window
    are given back, and a pool sized by ``pages_per_group`` never runs out."""
    from pyre_b200.cache import CacheManager, pages_for, pages_per_group
    kv = [KVGroup(PagedKVSpec(2, 16, window, keep_first=keep), 2), KVGroup(PagedKVSpec(1, 16, None), 1)]
    counts = pages_per_group(kv, page, 1000, max_requests=2, step_tokens=7)
    assert counts[1] == 1000 and counts[0] <= 2 * (pages_for(window + 6 + keep, page) + 2)
    m = CacheManager(kv, [], page, counts, 2, torch.float32, "cpu", allocate=False)
    length = {}
    rng = np.random.default_rng(page + keep)
    for r in ("a", "b", "c", "d"):          # two at a time; the later ones get the pages of the earlier ones
        m.begin(r)
        length[r] = 0
        if len(length) == 2:
            while any(n < 120 for n in length.values()):
                for q in list(length):
                    new = length[q] + int(rng.choice([1, 2, 7]))
                    assert m.reserve(q, new), f"a pool ran out at {new} tokens"
                    table = m.groups[0].tables[q]
                    for p in range(length[q], new):          # what this step's tokens read
                        seen = set(range(min(keep, p + 1))) | set(range(max(0, p - window + 1), p + 1))
                        assert all(table[j // page] >= 0 for j in seen)
                    m.commit(q, new)
                    length[q] = new
                m.check()
            for q in list(length):
                table = m.groups[0].tables[q]
                gone = range(pages_for(keep, page), max(0, length[q] - window + 1) // page)
                assert all(table[lp] == -1 for lp in gone) and len(gone) > 0
                m.end(q)
            length = {}
    assert m.stats().pages_free == m.stats().pages_total


def test_a_group_of_kept_tokens_is_its_own():
    kv = PagedKVSpec(2, 16, 32)
    assert kv != PagedKVSpec(2, 16, 32, keep_first=4) and PagedKVSpec(2, 16, 32, keep_first=4).tokens_held(8) == 31 + 8 + 4


def test_splits_are_planned_for_window_and_kept_tokens():
    from pyre_b200.parts.base import PartSpec, make_part
    part = make_part("mixer", PartSpec("attention", {"width": 64, "n_heads": 2, "n_kv_heads": 1, "head_dim": 64, "qkv_bias": False,
                                                     "window": 32, "keep_first": 4000}), torch.bfloat16, "cpu")
    near = make_part("mixer", PartSpec("attention", {"width": 64, "n_heads": 2, "n_kv_heads": 1, "head_dim": 64, "qkv_bias": False,
                                                     "window": 32}), torch.bfloat16, "cpu")
    assert part.launch_key(1, 8192) != near.launch_key(1, 8192) and part.launch_key(1, 20) == near.launch_key(1, 20)
    assert make_part("mixer", PartSpec("attention", {"width": 64, "n_heads": 2, "n_kv_heads": 1, "head_dim": 64, "qkv_bias": False,
                                                     "keep_first": 3}), torch.bfloat16, "cpu").cache_spec().keep_first == 0      # no window


# --------------------------------------------------------------------------- the host side through the replay loop
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for n, name in enumerate(["A", "B", "D"]):
        d = tmp_path_factory.mktemp(f"gad_{name}")
        raw = GH.GAD[name]
        GH.make_gadopel_dir(d, raw, seed=300 + n)
        reqs = {f"{name}{i}": GH.random_ids(raw, L, seed=17 * n + i) for i, L in enumerate([1, 2, 19, 37, 70])}
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
    GH.compare(_replay_on_cpu(monkeypatch, d, steps, GH.GAD_PAGE_SIZE[name]), plain, "float32", "portions")
    many = {f"{rid}r{rep}": ids for rep in range(2) for rid, ids in reqs.items()}     # ten requests, four alive at a time:
    steps = H.trace_mixed(many, seed=5, max_live=4)                                   # pages are used again
    got = _replay_on_cpu(monkeypatch, d, steps, GH.GAD_PAGE_SIZE[name])
    GH.compare(got, {f"{rid}r{rep}": plain[rid] for rep in range(2) for rid in reqs}, "float32", "mixed")


@pytest.mark.parametrize("fault", ["keep one more", "keep one fewer", "window one shorter", "no sink", "no second feed"])
def test_the_models_of_these_tests_show_a_fault(folders, monkeypatch, fault):
    """A mistake planted in the plain implementation moves its logits far beyond every bound used here."""
    d, reqs, plain = folders["A"]
    ids = reqs["A4"]
    if fault == "no sink":
        softmax = GP.softmax_sink
        monkeypatch.setattr(GP, "softmax_sink", lambda s, seen, sink=None: softmax(s, seen))
    elif fault == "no second feed":
        feed, seen = GP.feed_again, []
        monkeypatch.setattr(GP, "feed_again", lambda x, x0, w, lowp=False: (seen.append(1), feed(x, x0 if len(seen) < 2 else 0 * x0, w, lowp))[1])
    else:
        visible = GP.visible
        dk, dw = {"keep one more": (1, 0), "keep one fewer": (-1, 0), "window one shorter": (0, -1)}[fault]
        monkeypatch.setattr(GP, "visible", lambda T, window=None, keep=0: visible(T, window + dw, keep + dk) if window else visible(T))
    wrong = GH.plain_logits(d, ids)
    assert np.abs(wrong - plain["A4"]).max() > 30 * (1e-4 + 2e-4 * np.abs(plain["A4"]).max())


def test_a_layer_without_a_feed_forward_may_hold_its_second_norm(tmp_path, monkeypatch, folders):
    from safetensors.torch import load_file, save_file
    d, reqs, plain = folders["A"]
    state = load_file(str(d / "model.safetensors"))
    assert "l2.norm2" not in state
    state["l2.norm2"] = torch.full((96,), 3.0)
    (tmp_path / "config.json").write_text((d / "config.json").read_text())
    save_file(state, str(tmp_path / "model.safetensors"))
    got = _replay_on_cpu(monkeypatch, tmp_path, H.trace_whole({"A2": reqs["A2"]}), 16)
    GH.compare(got, {"A2": plain["A2"]}, "float32", "whole")


def test_random_model_folder_loads(tmp_path, monkeypatch):
    from pyre_b200.models.model import load_model
    from pyre_b200.weights import write_random_model

    standins.install(monkeypatch)
    cfg = config_from_dict(GH.GAD_D)
    write_random_model(tmp_path, cfg, seed=1)
    assert json.loads((tmp_path / "config.json").read_text())["architecture"] == "Gadopel"
    model, loaded = load_model(tmp_path, "cpu", "float32")
    assert loaded == cfg and model.loaded
    assert model.streams["loop.in"].w_x.shape == (128, 128) and model.streams["loop.in"].w_x0.is_contiguous()
