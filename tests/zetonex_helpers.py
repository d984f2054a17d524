"""Small Zetonex configurations and model folders for the tests. Tensor names and shapes are derived here from the
configuration, independently of the engine, so a folder written here also checks what the engine's loader expects.
Weights are drawn so that every mechanism carries weight in the logits: matrices of unit gain, norm weights and biases of order
one, lambdas well away from zero and one, tables that spread the tokens over all experts."""
from __future__ import annotations

import json
import random
from pathlib import Path
from typing import Dict, List, Sequence

import numpy as np
import torch
from safetensors.torch import save_file

import plain_zetonex as plain


def kept(heads, kv_heads, dim, scale=None, rot=0, base=10000.0, size=None, keep=0):
    """Sizes of the mixer whose values are its keys."""
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5 if scale is None else scale)
    if rot:
        m["rot"] = dict(base=base, dims=rot)
    if size is not None:
        m["mask"] = dict(size=size, keep_first=keep)
    return m


def scaling(factor, low, high, original):
    return dict(factor=factor, low=low, high=high, original=original)


def difference(heads, kv_heads, dim, vdim, scale=None, rot=0, base=10000.0, size=None, diff=0.3, softcap=None, blend=None):
    """Sizes of the differential mixer; ``blend``: the rotation's frequency scaling."""
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=dim ** -0.5 if scale is None else scale, diff=diff)
    if rot:
        m["rot"] = dict(base=base, dims=rot)
        if blend is not None:
            m["rot"]["scaling"] = blend
    if size is not None:
        m["mask"] = dict(size=size)
    if softcap is not None:
        m["softcap"] = softcap
    return m


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, limit=0.8):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))


def layer(kind, mixer, mlp=None):
    return dict(type=kind, mixer=mixer, mlp=mlp)


def config(layers, vocab=300, width=72, eps=1e-5, logit_scale=0.6, loop=None):
    c = dict(architecture="Zetonex", vocab=vocab, width=width, norm=dict(eps=eps), logit_scale=logit_scale, layers=layers)
    if loop is not None:
        c["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return c


def _mix():
    """Odd sizes everywhere, keys and values of different sizes, a stretch in the middle that runs three times."""
    return config([
        layer("attention_2", difference(6, 2, 10, 28, scale=0.4, rot=6, size=19, diff=0.45, softcap=3.0), dense(56)),
        layer("attention", kept(6, 3, 20, scale=0.3, rot=12, size=7, keep=5), moe(5, 3, 24, limit=0.7)),
        layer("attention_2", difference(4, 4, 12, 24, scale=0.5, rot=12, base=500.0, size=11, diff=0.2,
                                        blend=scaling(6.0, 1.0, 5.0, 90)), moe(7, 1, 16, limit=1.5)),
        layer("attention", kept(3, 1, 12, scale=0.5, rot=4, size=16, keep=9), None),
        layer("attention", kept(4, 2, 16, scale=0.4, rot=16, base=200.0, size=5, keep=1), dense(40)),
    ], loop=(1, 3, 3))


def _wide():
    """Sizes that reach the tensor-core products and attention kernels; the loop starts at the first layer."""
    return config([
        layer("attention", kept(4, 2, 64, scale=0.2, rot=32, base=1e6, size=50, keep=3), moe(8, 3, 64)),
        layer("attention_2", difference(4, 2, 32, 64, scale=0.25, rot=16, size=70, diff=0.6, softcap=5.0,
                                        blend=scaling(3.0, 2.0, 3.0, 300)), dense(136)),
        layer("attention_2", difference(2, 1, 64, 128, scale=0.2, rot=64, size=90, diff=0.1), moe(6, 2, 64, limit=2.0)),
        layer("attention", kept(4, 4, 128, scale=0.09, rot=64, size=33, keep=20), dense(128)),
    ], vocab=515, width=128, eps=1e-6, logit_scale=1.3, loop=(0, 2, 2))


def _one():
    """One of everything: one head, windows of one and two keys, one kept position or none, one expert, a loop that runs once;
    no mask, no rotation, no cap in some layers; factors of one."""
    return config([
        layer("attention", kept(1, 1, 8, rot=8, size=1, keep=1), moe(1, 1, 16, limit=1.0)),
        layer("attention_2", difference(3, 1, 8, 8, rot=2, size=1, diff=0.0), None),
        layer("attention", kept(2, 1, 16, size=2, keep=0), moe(3, 3, 8)),
        layer("attention_2", difference(1, 1, 4, 40, scale=1.0, diff=0.5, softcap=1.0), dense(8)),
        layer("attention", kept(2, 2, 8, scale=1.0, rot=4), None),
    ], width=40, logit_scale=1.0, loop=(2, 3, 1))


MIX, WIDE, ONE = _mix(), _wide(), _one()


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W = cfg["width"]
    shapes = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": (W,)}
    if cfg.get("loop"):
        shapes["loop.in"] = (W, 2 * W)
    for i, entry in enumerate(cfg["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        shapes[p + "norm1"] = (W,)
        shapes[p + "mix.o"] = (W, H * dv)
        if entry["type"] == "attention":
            shapes.update({p + "mix.q": (H * d, W), p + "mix.k": (G * d, W), p + "mix.g": (H * dv, W)})
        else:
            shapes.update({p + "mix.q": (H * 2 * d, W), p + "mix.k": (G * 2 * d, W), p + "mix.v": (G * dv, W)})
            for name in ("q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2"):
                shapes[p + "mix." + name] = (d,)
        f = entry.get("mlp")
        if f is None:
            continue
        if f["kind"] == "dense":
            for name, rows, cols in (("gate", f["ff"], W), ("up", f["ff"], W), ("down", W, f["ff"])):
                shapes.update({p + "mlp." + name: (rows, cols), p + f"mlp.{name}.b": (rows,)})
            continue
        ff = f["expert"]["ff"]
        for e in range(f["router"]["experts"]):
            shapes.update({p + f"mlp.e{e}.gate": (ff, W), p + f"mlp.e{e}.up": (ff, W), p + f"mlp.e{e}.down": (W, ff)})
        shapes[p + "mlp.table"] = (cfg["vocab"], f["router"]["top"])
    return shapes


def draw_tensors(cfg: dict, seed: int, dtype=torch.float32) -> Dict[str, torch.Tensor]:
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[1] if name.startswith("l") else name
        if leaf == "mlp.table":
            experts = cfg["layers"][int(name.split(".")[0][1:])]["mlp"]["router"]["experts"]
            out[name] = torch.rand(shape[0], experts, generator=gen).argsort(-1)[:, :shape[1]].to(torch.int32).contiguous()
            continue
        t = torch.randn(shape, generator=gen, dtype=torch.float32)
        if leaf == "norm1" or name == "final.norm":
            t = 0.3 * t
        elif leaf in ("mix.q.norm", "mix.k.norm"):
            t = 1.0 + 0.2 * t
        elif leaf in ("mix.lq1", "mix.lk1", "mix.lq2", "mix.lk2"):
            t = 0.5 * t
        elif leaf.endswith(".b"):
            t = 0.5 * t
        elif name != "embed":
            t = t / shape[-1] ** 0.5                     # unit gain
        out[name] = t.to(dtype).contiguous()
    return out


def write_folder(folder, cfg: dict, seed: int, dtype: str = "float32", edit=None) -> Path:
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    tensors = draw_tensors(cfg, seed, torch.float32 if dtype == "float32" else torch.bfloat16)
    if edit is not None:
        edit(tensors)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file(tensors, str(folder / "model.safetensors"))
    return folder


def read_folder(folder):
    from safetensors.torch import load_file
    cfg = json.loads((Path(folder) / "config.json").read_text())
    return cfg, load_file(str(Path(folder) / "model.safetensors"))


def random_requests(cfg: dict, lengths: Sequence[int], seed: int) -> Dict[str, List[int]]:
    rng = random.Random(seed)
    return {f"r{i}": [rng.randrange(cfg["vocab"]) for _ in range(n)] for i, n in enumerate(lengths)}


def forward(cfg, w, tokens, residuals=None) -> np.ndarray:
    return plain.Model(cfg, w, torch.float64).run(tokens, residuals=residuals).numpy()


def plain_logits(folder, requests) -> Dict[str, np.ndarray]:
    cfg, w = read_folder(folder)
    return {rid: forward(cfg, w, toks) for rid, toks in requests.items()}
