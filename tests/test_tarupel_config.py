"""The Tarupel design on the CPU: configuration, tensor names and shapes, run order, cache entries and state, refused
configurations, the random-weights folder, pages that a chunk has passed, and the plain statement against itself (the
premises of the GPU tests: what a mask one key off, a forgotten shift or a group left in the choice does to the logits)."""
import copy

import numpy as np
import pytest
import torch

import plain_tarupel as plain
import tarupel_helpers as th
from tinyinfer_b200 import models  # noqa: F401
from tinyinfer_b200.cache import CacheManager
from tinyinfer_b200.config import TarupelConfig, load_config, lookup_architecture, preset_config
from tinyinfer_b200.parts.base import CacheNeed
from tinyinfer_b200.weights import load_weights, write_random_model


def build(cfg):
    return lookup_architecture("Tarupel").model_factory(TarupelConfig.from_dict(cfg), torch.float32, "cpu")


@pytest.mark.parametrize("name", ["MIX", "WIDE", "ONE"])
def test_names_and_shapes_follow_the_configuration(name, tmp_path):
    cfg = getattr(th, name)
    want = th.tensor_shapes(cfg)
    model = build(cfg)
    got = model.expected_tensors()
    assert set(got) == set(want)
    assert {n: tuple(ts.shape) for n, ts in got.items()} == want
    # the inner size of the decay's projections need not stand in the configuration: it is the checkpoint's
    bare = copy.deepcopy(cfg)
    for l in bare["layers"]:
        l["mixer"].pop("gate_rank", None)
    folder = th.write_folder(tmp_path / "m", cfg, seed=1)
    loaded = build(bare)
    load_weights(loaded, folder)
    norm = loaded.blocks[0].mixer_norm.as_rms()[0]
    stored = th.read_folder(folder)[1]["l0.norm1"]
    assert stored.dim() == 0 and norm.shape == (cfg["width"],) and bool((norm == stored).all())


def test_run_order_cache_entries_and_state():
    model = build(th.MIX)
    order = [(e.layer, e.cache, e.adds_embedding, e.adds_vector) for e in model.spec.execution]
    assert order == [(0, 0, False, None), (1, 1, False, 0), (2, 2, False, None), (1, 3, True, 1), (2, 4, False, None),
                     (1, 5, True, 2), (2, 6, False, None), (3, 7, False, None), (4, 8, False, None), (5, 9, False, None)]
    W, needs = th.MIX["width"], model.cache_needs()
    assert len(needs) == 10
    # every run keeps the token before in its slot, behind the mixer's own state: a convolution's inputs, a matrix per head
    states = [s.shape[0] - W for _, s in needs]
    assert states == [2 * (120 + 40 + 24), 432, 0, 432, 0, 432, 0, 800, 0, 4 * 72]
    kv = [(n.num_kv_heads, n.head_dim, n.window, n.chunk, n.planes) if n else None for n, _ in needs]
    assert kv[0] == (2, 32, None, 19, 1) and kv[2] == (4, 16, 11, None, 2) and kv[1] is None and kv[8] == (3, 32, 5, None, 1)
    assert kv[4] == kv[2] and kv[9] == (3, 8, None, 7, 2)
    plain_order = plain.run_order(th.MIX)
    assert [(i, t) for i, t in plain_order] == [(e.layer, e.adds_vector) for e in model.spec.execution]
    without = copy.deepcopy(th.MIX)
    del without["loop"]
    spec = build(without).spec
    assert spec.step_vectors is None and [e.layer for e in spec.execution] == list(range(6))


def test_constants_reach_the_specs():
    spec = build(th.MIX).spec
    l0, l1, l2 = spec.layers[:3]
    assert all(l.arrangement == "scaled_residual" and l.residual_mult == 0.8 and l.token_shift == "shift" for l in spec.layers)
    assert l0.mixer_norm.single_gain and l0.mixer_norm.eps == 1e-5
    a = l0.mixer
    assert (a.conv_taps, a.chunk, a.window, a.qk_unit_norm, a.qkv_bias, a.scale) == (3, 19, None, 1e-5, True, 0.3)
    assert not a.position.interleaved and a.position.rotary_dim == 12 and a.position.theta == 10000.0
    d = l1.mixer
    assert (d.num_heads, d.key_dim, d.value_dim, d.unit_eps) == (3, 12, 12, 1e-6) and abs(d.decay_scale + 0.6065306597126334) < 1e-15
    moe = l1.feed_forward
    assert (moe.num_experts, moe.top, moe.groups, moe.keep_groups, moe.weight_scale, moe.shared_size, moe.shared_gate) == \
        (6, 3, 3, 2, 1.7, 40, True)
    assert moe.scoring == "softmax" and moe.renormalize and moe.router_input == "input" and moe.activation == "silu_glu"
    b = l2.mixer
    assert (b.window, b.chunk, b.conv_taps, b.qk_row_norm.eps, b.qkv_bias) == (11, None, 0, 1e-5, True) and b.position.interleaved
    assert l0.feed_forward.activation == "gelu_tanh" and spec.layers[3].feed_forward is None
    plain_moe = spec.layers[4].feed_forward
    assert (plain_moe.groups, plain_moe.keep_groups, plain_moe.shared_size, plain_moe.shared_gate) == (1, 1, 0, False)


@pytest.mark.parametrize("edit,message", [
    (lambda c: c["layers"][0].update(type="chunked"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("dim"), "lacks mixer.dim"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22), "dims even and at most dim"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "at least 1"),
    (lambda c: c["layers"][0]["mixer"].update(conv=-1), "not be negative"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "exceeds the experts"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "equal groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "equal groups"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("ff"), "shared.ff"),
    (lambda c: c["layers"][0]["mlp"].update(kind="wide"), "unknown feed-forward"),
    (lambda c: c["loop"].update(stop=7), "stretch of the layers"),
    (lambda c: c["loop"].pop("times"), "start, stop and times"),
    (lambda c: c.pop("norm"), "required keys"),
])
def test_refused_configurations(edit, message):
    cfg = copy.deepcopy(th.MIX)
    edit(cfg)
    with pytest.raises(ValueError, match=message):
        TarupelConfig.from_dict(cfg)


def test_round_trip_presets_and_random_folder(tmp_path):
    cfg = TarupelConfig.from_dict(th.MIX)
    assert TarupelConfig.from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    tiny = preset_config("tarupel-tiny")
    folder = write_random_model(tmp_path / "r", tiny, seed=1)
    arch, again = load_config(folder)
    assert arch.name == "Tarupel" and again.to_dict() == tiny.to_dict()
    from safetensors.torch import load_file
    stored = load_file(str(folder / "model.safetensors"))
    assert {n: tuple(t.shape) for n, t in stored.items()} == th.tensor_shapes(tiny.to_dict())
    for preset in ("tarupel-1b", "tarupel-2b"):
        assert build(preset_config(preset).to_dict()).weight_bytes() > 5e8


def test_a_frame_without_a_residual_to_add_to_refuses():
    from tinyinfer_b200.models import DecoderModel
    from tinyinfer_b200.config import ExecStep
    with pytest.raises(NotImplementedError, match="no residual"):
        DecoderModel.enter(object.__new__(DecoderModel), None, ExecStep(0, 0, adds_embedding=True))
    with pytest.raises(ValueError, match="adds a vector"):
        import dataclasses
        dataclasses.replace(build(th.ONE).spec, step_vectors=None)


@pytest.mark.parametrize("chunk,page", [(19, 4), (8, 8), (5, 16), (64, 16)])
def test_pages_of_a_passed_chunk_are_given_back(chunk, page):
    """A request that grows token by token never lacks a page of its own chunk, and holds none that only earlier chunks
    need; the pool is far smaller than the request is long."""
    need = CacheNeed(1, 8, chunk=chunk)
    assert not need.keeps_all and need.first_read(chunk - 1) == 0 and need.first_read(chunk) == chunk
    manager = CacheManager([(need, None)], page, (chunk + page - 1) // page + 1, 1)
    manager.admit("a")
    for n in range(1, 4 * chunk + 40):
        manager.extend("a", n)
        table, first = manager.get("a").tables[0], (n - 1) // chunk * chunk
        assert all(table[i] >= 0 for i in range(first // page, (n - 1) // page + 1)), n
        manager.commit("a", n)
        manager.check_consistency()
        assert sum(t >= 0 for t in manager.get("a").tables[0]) <= (chunk + page - 1) // page + 1
    manager.release("a")
    manager.check_consistency()
    assert manager.stats()["groups"][0]["free_pages"] == (chunk + page - 1) // page + 1


# ------------------------------------------------------------------ the plain statement against itself
def quiet(t):
    """No token shift and a convolution of the current token alone: a key then hangs on its own token only."""
    for name in t:
        if name.endswith(".shift"):
            t[name] = torch.zeros_like(t[name])
        if name.endswith(".conv"):
            t[name] = torch.zeros_like(t[name])
            t[name][:, -1] = 1.0
    return t


@pytest.mark.parametrize("kind,inside,outside", [("attention", 24, 23), ("attention_2", 24, 23)])
def test_plain_masks_are_exact_to_the_key(kind, inside, outside):
    """Position 29 of chunks of 8 sees 24 .. 29; behind a window of 6 it sees 24 .. 29 too."""
    size = 8 if kind == "attention" else 6
    cfg = th.config([th.layer(kind, th.attention(2, 1, 8, 12, rot=8, size=size, conv=3 if kind == "attention" else 0), None)], width=32)
    w = quiet(th.draw_tensors(cfg, 3, torch.float64))
    tokens = th.random_requests(cfg, [30], seed=1)["r0"]
    base = th.forward(cfg, w, tokens)

    def moved(p):
        other = list(tokens)
        other[p] = (other[p] + 1) % cfg["vocab"]
        return np.abs(th.forward(cfg, w, other)[29] - base[29]).max()
    assert moved(outside) == 0.0 and moved(inside) > 1e-3 * np.abs(base).max()


def test_plain_mechanisms_carry_weight():
    """Leaving one mechanism out of the plain statement moves the logits far beyond the GPU tests' tolerances."""
    cfg = th.MIX
    w = th.draw_tensors(cfg, 5, torch.float64)
    tokens = th.random_requests(cfg, [40], seed=2)["r0"]
    base = th.forward(cfg, w, tokens)
    scale = np.abs(base).max()

    def moved(edit_cfg=None, edit_w=None):
        c, t = copy.deepcopy(cfg), dict(w)
        if edit_cfg:
            edit_cfg(c)
        if edit_w:
            edit_w(t)
        return np.abs(th.forward(c, t, tokens) - base).max() / scale

    def zeroed(*names):
        return lambda t: t.update({n: torch.zeros_like(t[n]) for n in names})

    def ones(*names):
        return lambda t: t.update({n: torch.ones_like(t[n]) for n in names})
    for i in (0, 2, 4, 5):
        assert moved(lambda c: c["layers"][i]["mixer"]["mask"].update(size=c["layers"][i]["mixer"]["mask"]["size"] + 1)) > 1e-3, i
    assert moved(lambda c: c["loop"].update(times=2)) > 1e-2
    assert moved(lambda c: c.update(residual_mult=0.79)) > 1e-3
    assert moved(lambda c: c["layers"][1]["mlp"]["router"].update(groups=dict(count=3, keep=3))) > 1e-3
    assert moved(lambda c: c["layers"][4]["mlp"]["router"].update(scale=1.0)) > 1e-3
    assert moved(lambda c: c["layers"][0]["mixer"].pop("rot")) > 1e-3 and moved(lambda c: c["layers"][2]["mixer"].pop("rot")) > 1e-3
    for i in range(6):
        assert moved(edit_w=zeroed(f"l{i}.shift")) > 1e-2, i
        assert moved(edit_w=ones(f"l{i}.ls1")) > 1e-3 and moved(edit_w=ones(f"l{i}.norm1")) > 1e-4, i
    assert moved(edit_w=zeroed("loop.step")) > 1e-2 and moved(edit_w=zeroed("l0.mix.k.b")) > 1e-3
    assert moved(edit_w=zeroed("l1.mix.w2")) > 1e-3 and moved(edit_w=zeroed("l1.mix.a")) > 1e-3
    assert moved(edit_w=zeroed("l1.mlp.shared.sg")) > 1e-3 and moved(edit_w=ones("l2.mix.q.norm")) > 1e-3


def test_plain_group_choice():
    """The best two experts overall may lie in a group that is not kept."""
    scores = torch.tensor([0.30, 0.01, 0.02, 0.29, 0.05, 0.26, 0.03, 0.04])      # groups of two: bests .30 .29 .26 .04
    assert sorted(plain.grouped_choice(scores, 3, 4, 2).tolist()) == [0, 2, 3]
    assert sorted(plain.grouped_choice(scores, 3, 1, 1).tolist()) == [0, 3, 5]
    assert sorted(plain.grouped_choice(scores, 2, 4, 1).tolist()) == [0, 1]


def test_plain_delta_rule_replaces_and_decays():
    """Unit rate, no decay, a unit key written twice: a reader along it gets the second value alone; at rate 0 both add up;
    a decay acts on a key channel whatever its rate."""
    e0 = torch.tensor([[[1.0, 0.0, 0.0]]], dtype=torch.float64)
    k, r = e0.repeat(2, 1, 1), e0.repeat(2, 1, 1)
    v = torch.tensor([[[2.0, 3.0]], [[5.0, -7.0]]], dtype=torch.float64)
    one = torch.ones(2, 1, 3, dtype=torch.float64)
    o, S = plain.general_delta_rule(r, k, v, one, one, torch.zeros(1, 3, 2, dtype=torch.float64))
    assert torch.allclose(o[1], v[1], atol=1e-5) and torch.allclose(S[0, 0], v[1, 0], atol=1e-5)
    o, _ = plain.general_delta_rule(r, k, v, one, 0 * one, torch.zeros(1, 3, 2, dtype=torch.float64))
    assert torch.allclose(o[1], v[0] + v[1])
    o, _ = plain.general_delta_rule(r, k, v, 0.5 * one, 0 * one, torch.zeros(1, 3, 2, dtype=torch.float64))
    assert torch.allclose(o[1], 0.5 * v[0] + v[1])
