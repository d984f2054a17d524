"""The Zetonex design on the CPU: configuration, tensor names and shapes, run order, cache entries, refused configurations, the
random-weights folder, pages that a window has passed beside those of kept first positions, and the plain statement against
itself (the premises of the GPU tests: what a mask one key off, a kept position too few or a forgotten gate does to the
logits)."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_zetonex as plain
import zetonex_helpers as zh
from tinyinfer_b200 import models  # noqa: F401
from tinyinfer_b200.cache import CacheManager
from tinyinfer_b200.config import ZetonexConfig, load_config, lookup_architecture, preset_config
from tinyinfer_b200.config.specs import PositionSpec, WavelengthBlend
from tinyinfer_b200.parts.base import CacheNeed, build_position
from tinyinfer_b200.weights import load_weights, write_random_model


def build(cfg):
    return lookup_architecture("Zetonex").model_factory(ZetonexConfig.from_dict(cfg), torch.float32, "cpu")


@pytest.mark.parametrize("name", ["MIX", "WIDE", "ONE"])
def test_names_and_shapes_follow_the_configuration(name, tmp_path):
    cfg = getattr(zh, name)
    model = build(cfg)
    assert {n: tuple(ts.shape) for n, ts in model.expected_tensors().items()} == zh.tensor_shapes(cfg)
    folder = zh.write_folder(tmp_path / "m", cfg, seed=1)
    load_weights(model, folder)
    w = zh.read_folder(folder)[1]
    # a weight stored around zero; a factor on the logits that rides in the final norm; one lambda a differential layer
    assert torch.equal(model.blocks[0].mixer_norm.as_rms()[0], w["l0.norm1"] + 1.0)
    assert torch.allclose(model._logit_norm, (w["final.norm"] + 1.0) * cfg["logit_scale"])
    for i, entry in enumerate(cfg["layers"]):
        if entry["type"] == "attention_2":
            sub = {k[len(f"l{i}.mix."):]: v.double() for k, v in w.items() if k.startswith(f"l{i}.mix.")}
            assert abs(model.blocks[i].mixer.share - plain.difference_share(sub, entry["mixer"]["diff"])) < 1e-12
    assert torch.equal(model.entry_weight, w["loop.in"])


def test_a_bfloat16_model_projects_both_halves_of_the_residual(tmp_path):
    folder = zh.write_folder(tmp_path / "m", zh.ONE, seed=1, dtype="bfloat16")
    model = lookup_architecture("Zetonex").model_factory(ZetonexConfig.from_dict(zh.ONE), torch.bfloat16, "cpu")
    load_weights(model, folder)
    w, W = zh.read_folder(folder)[1]["loop.in"], zh.ONE["width"]
    assert torch.equal(model.entry_weight, torch.cat([w[:, :W], w[:, :W], w[:, W:]], dim=1))


def test_run_order_and_cache_entries():
    model = build(zh.MIX)
    order = [(e.layer, e.cache, e.projects_embedding) for e in model.spec.execution]
    assert order == [(0, 0, False), (1, 1, True), (2, 2, False), (1, 3, True), (2, 4, False), (1, 5, True), (2, 6, False),
                     (3, 7, False), (4, 8, False)]
    assert [(i, s) for i, s in plain.run_order(zh.MIX)] == [(e.layer, e.projects_embedding) for e in model.spec.execution]
    needs = model.cache_needs()
    assert all(state is None for _, state in needs) and len(needs) == 9
    kv = [(n.num_kv_heads, n.head_dim, n.window, n.keep_first, n.planes) for n, _ in needs]
    assert kv[0] == (2, 48, 19, 0, 1)                   # a key of two maps of 10 and a value of 28 in one row
    assert kv[1] == kv[3] == kv[5] == (3, 20, 7, 5, 2)
    assert kv[2] == kv[6] == (4, 24, 11, 0, 2)          # two maps of 12 are as long as a value: two planes
    assert kv[8] == (2, 16, 5, 1, 2)
    without = copy.deepcopy(zh.MIX)
    del without["loop"]
    spec = build(without).spec
    assert spec.entry_projection is None and [e.layer for e in spec.execution] == list(range(5))


def test_constants_reach_the_specs():
    spec = build(zh.MIX).spec
    l0, l1, l2, l3, _ = spec.layers
    assert all(l.arrangement == "parallel_residual" and l.feed_forward_norm is None and l.mixer_norm.offset == 1.0 for l in spec.layers)
    a = l0.mixer
    assert (a.maps, a.difference, a.difference_eps, a.softcap, a.window, a.scale, a.v_dim) == (2, 0.45, 1e-5, 3.0, 19, 0.4, 28)
    assert a.qk_norm.size == 10 and a.qk_norm.offset == 0.0 and not a.values_are_keys and not a.feature_gate
    assert (a.q_size, a.kv_size) == (120, 40)
    b = l1.mixer
    assert (b.maps, b.values_are_keys, b.feature_gate, b.keep_first, b.window, b.softcap) == (1, True, True, 5, 7, None)
    assert (b.position.rotary_dim, b.position.theta, b.position.interleaved) == (12, 10000.0, False) and b.qk_norm is None
    assert l2.mixer.position.blend == WavelengthBlend(6.0, 1.0, 5.0, 90.0)
    f = l1.feed_forward
    assert (f.num_experts, f.top, f.expert_size, f.glu_limit, f.glu_alpha, f.table_rows) == (5, 3, 24, 0.7, 1.702, 300)
    assert l0.feed_forward.bias and l0.feed_forward.activation == "silu" and l3.feed_forward is None


@pytest.mark.parametrize("edit,message", [
    (lambda c: c["layers"][0].update(type="differential"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "lacks mixer.diff"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=24), "the keys' size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=12), "dims even and at most dim"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("low"), "factor, low, high and original"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "at least 1"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1), "not negative"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=0.0), "softcap must be positive"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "number of experts"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "expert.limit"),
    (lambda c: c["layers"][0]["mlp"].update(kind="wide"), "unknown feed-forward"),
    (lambda c: c["loop"].update(stop=6), "stretch of the layers"),
    (lambda c: c["loop"].pop("times"), "start, stop and times"),
    (lambda c: c.pop("norm"), "required keys"),
])
def test_refused_configurations(edit, message):
    cfg = copy.deepcopy(zh.MIX)
    edit(cfg)
    with pytest.raises(ValueError, match=message):
        ZetonexConfig.from_dict(cfg)


def test_a_table_that_names_no_expert_is_refused(tmp_path):
    folder = zh.write_folder(tmp_path / "m", zh.ONE, seed=1, edit=lambda t: t["l0.mlp.table"].fill_(1))
    with pytest.raises(ValueError, match="outside 0..0"):
        load_weights(build(zh.ONE), folder)


def test_round_trip_presets_and_random_folder(tmp_path):
    cfg = ZetonexConfig.from_dict(zh.MIX)
    assert ZetonexConfig.from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    tiny = preset_config("zetonex-tiny")
    folder = write_random_model(tmp_path / "r", tiny, seed=1)
    arch, again = load_config(folder)
    assert arch.name == "Zetonex" and again.to_dict() == tiny.to_dict()
    from safetensors.torch import load_file
    stored = load_file(str(folder / "model.safetensors"))
    assert {n: tuple(t.shape) for n, t in stored.items()} == zh.tensor_shapes(tiny.to_dict())
    table = stored["l1.mlp.table"]
    assert table.dtype == torch.int32 and int(table.min()) == 0 and int(table.max()) == 5 and bool((table[:, 0] != table[:, 1]).all())
    for preset in ("zetonex-1b", "zetonex-2b"):
        assert build(preset_config(preset).to_dict()).weight_bytes() > 5e8


@pytest.mark.parametrize("window,keep,page", [(7, 5, 4), (8, 8, 8), (5, 1, 16), (33, 20, 16), (1, 3, 4), (6, 0, 4)])
def test_pages_behind_a_window_go_back_and_those_of_kept_positions_stay(window, keep, page):
    """A request that grows token by token never lacks a page it may read, and holds none that nobody reads; the pool is
    smaller than the request is long."""
    need = CacheNeed(1, 8, window=window, keep_first=keep)
    most = (keep + page - 1) // page + (window + page - 1) // page + 1
    manager = CacheManager([(need, None)], page, most, 1)
    manager.admit("a")
    for n in range(1, 6 * window + keep + 5 * page):
        manager.extend("a", n)
        table, lo = manager.get("a").tables[0], max(0, n - window)
        seen = [p for p in range(n) if p >= lo or p < keep]
        assert all(table[p // page] >= 0 for p in seen), n
        manager.commit("a", n)
        manager.check_consistency()
        after = {p // page for p in range(n + 1) if p >= n + 1 - window or p < keep}
        assert all(table[i] < 0 or i in after for i in range(len(table))), n
    manager.release("a")
    manager.check_consistency()
    assert manager.stats()["groups"][0]["free_pages"] == most


@pytest.mark.parametrize("blend", [None, (5.0, 1.0, 4.0, 400), (8.0, 2.0, 2.0, 100), (2.0, 1.0, 8.0, 64)])
def test_frequencies_scaled_by_wavelength(blend):
    """Against the plain statement, pair by pair; the middle range is reached where there is one."""
    rot = dict(base=5000.0, dims=32)
    spec = None
    if blend:
        rot["scaling"] = zh.scaling(*blend)
        spec = WavelengthBlend(*(float(b) for b in blend))
    part = build_position(PositionSpec(kind="rope", theta=5000.0, rotary_dim=32, exact_frequencies=True, blend=spec), torch.float32, "cpu")
    want = plain.frequencies(rot)
    assert torch.equal(part.inv_freq, want.to(torch.float32))
    free = plain.frequencies(dict(base=5000.0, dims=32))
    if blend:
        slowed, untouched = want == free / blend[0], want == free
        assert bool(slowed.any()) and bool(untouched.any())
        if blend[2] > blend[1]:
            assert bool((~slowed & ~untouched).any())


# ------------------------------------------------------------------ the plain statement against itself
def test_plain_masks_are_exact_to_the_key():
    """Position 29 behind a window of 6 with 3 kept positions sees 0 .. 2 and 24 .. 29."""
    for kind, mixer, kept in (("attention", zh.kept(2, 1, 8, rot=8, size=6, keep=3), 3), ("attention_2", zh.difference(2, 1, 8, 12, size=6), 0)):
        cfg = zh.config([zh.layer(kind, mixer, None)], width=32)
        w = zh.draw_tensors(cfg, 3, torch.float64)
        tokens = zh.random_requests(cfg, [30], seed=1)["r0"]
        base = zh.forward(cfg, w, tokens)

        def moved(p):
            other = list(tokens)
            other[p] = (other[p] + 1) % cfg["vocab"]
            return np.abs(zh.forward(cfg, w, other)[29] - base[29]).max() / np.abs(base).max()
        for p in range(29):
            assert (moved(p) > 1e-5) == (p >= 24 or p < kept) and (p >= 24 or p < kept or moved(p) == 0.0), (kind, p)


def test_plain_mechanisms_carry_weight():
    """Leaving one mechanism out of the plain statement moves the logits far beyond the GPU tests' tolerances."""
    cfg = zh.MIX
    w = zh.draw_tensors(cfg, 5, torch.float64)
    tokens = zh.random_requests(cfg, [40], seed=2)["r0"]
    base = zh.forward(cfg, w, tokens)
    scale = np.abs(base).max()

    def moved(edit_cfg=None, edit_w=None):
        c, t = copy.deepcopy(cfg), dict(w)
        if edit_cfg:
            edit_cfg(c)
        if edit_w:
            edit_w(t)
        return np.abs(zh.forward(c, t, tokens) - base).max() / scale

    def set_mixer(i, **kw):
        return lambda c: c["layers"][i]["mixer"].update(**kw)

    def zeroed(*names):
        return lambda t: t.update({n: torch.zeros_like(t[n]) for n in names})
    for i in range(5):
        mask = cfg["layers"][i]["mixer"]["mask"]
        assert moved(set_mixer(i, mask=dict(mask, size=mask["size"] + 1))) > 1e-3, i
        assert moved(lambda c: c["layers"][i]["mixer"].pop("rot")) > 1e-3, i
        assert moved(edit_w=zeroed(f"l{i}.norm1")) > 1e-2, i
        if cfg["layers"][i]["type"] == "attention":
            assert moved(set_mixer(i, mask=dict(mask, keep_first=mask["keep_first"] - 1))) > 1e-3, i
            assert moved(set_mixer(i, mask=dict(mask, keep_first=mask["keep_first"] + 1))) > 1e-3, i
            assert moved(edit_w=zeroed(f"l{i}.mix.g")) > 1e-2, i
        else:
            assert moved(set_mixer(i, diff=cfg["layers"][i]["mixer"]["diff"] + 0.05)) > 1e-3, i
            assert moved(edit_w=zeroed(f"l{i}.mix.lq1")) > 1e-3 and moved(edit_w=zeroed(f"l{i}.mix.lk2")) > 1e-3, i
            assert moved(edit_w=lambda t: t.update({f"l{i}.mix.q.norm": torch.ones_like(t[f"l{i}.mix.q.norm"])})) > 1e-3, i
    assert moved(lambda c: c["layers"][0]["mixer"].pop("softcap")) > 1e-3
    assert moved(lambda c: c["layers"][2]["mixer"]["rot"].pop("scaling")) > 1e-3
    assert moved(lambda c: c["loop"].update(times=2)) > 1e-2 and moved(lambda c: c.update(logit_scale=0.59)) > 1e-3
    W = cfg["width"]
    assert moved(edit_w=lambda t: t.update({"loop.in": torch.cat([t["loop.in"][:, :W], 0 * t["loop.in"][:, W:]], dim=1)})) > 1e-2
    for limit, i in ((1e3, 1), (1e3, 2)):
        assert moved(lambda c: c["layers"][i]["mlp"]["expert"].update(limit=limit)) > 1e-3, i
    assert moved(edit_w=lambda t: t.update({"l1.mlp.table": (t["l1.mlp.table"] + 1) % 5})) > 1e-2
    for name in ("gate", "up", "down"):
        assert moved(edit_w=zeroed(f"l0.mlp.{name}.b")) > 1e-3, name


def test_plain_difference_of_equal_maps():
    """With both maps alike the difference is (1 - lambda) times one map, and the norm takes the factor away."""
    d, dv, T, eps = 6, 10, 9, 1e-12
    gen = torch.Generator().manual_seed(0)
    w = {n: torch.randn(s, generator=gen, dtype=torch.float64) for n, s in
         (("q", (2 * d, 16)), ("k", (2 * d, 16)), ("v", (dv, 16)), ("o", (dv, dv)), ("q.norm", (d,)), ("k.norm", (d,)))}
    w["q"][d:], w["k"][d:] = w["q"][:d], w["k"][:d]
    w.update({n: torch.zeros(d, dtype=torch.float64) for n in ("lq1", "lk1", "lq2", "lk2")})
    m = zh.difference(1, 1, d, dv, size=4, diff=0.3)
    H = torch.randn(T, 16, generator=gen, dtype=torch.float64)
    assert abs(plain.difference_share(w, 0.3) - 0.3) < 1e-15
    q, k = ((plain.rms(H @ w[n][:d].t(), eps) * w[n + ".norm"]) for n in ("q", "k"))
    one = plain.softmax_weights(q, k, m["scale"], plain.seen(T, 4)) @ (H @ w["v"].t())
    assert torch.allclose(plain.differential_attention(w, m, eps, H), 0.7 * plain.rms(one, eps) @ w["o"].t())


def test_plain_scaled_frequency_meets_at_both_ends():
    """At the two wavelengths where the ranges meet, the blend equals what the range beyond it gives."""
    s = zh.scaling(5.0, 1.5, 6.0, 400)
    for length, want in ((400 / 6.0, 1.0), (400 / 1.5, 0.2)):
        share = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
        assert math.isclose((1 - share) / s["factor"] + share, want)
