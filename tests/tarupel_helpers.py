"""Small Tarupel configurations and model folders for the tests. Tensor names and shapes are derived here from the
configuration, independently of the engine, so a folder written here also checks what the engine's loader expects.
Weights are drawn so that every mechanism carries weight in the logits: matrices of unit gain, scales and shifts of order
one, decays and removal rates spread over their ranges, router rows large enough that the scores differ."""
from __future__ import annotations

import json
import random
from pathlib import Path
from typing import Dict, List, Sequence

import numpy as np
import torch
from safetensors.torch import save_file

import plain_tarupel as plain


def attention(heads, kv_heads, dim, vdim, scale=None, rot=0, base=10000.0, size=None, conv=0):
    """Sizes of either attention; ``conv`` only means something for 'attention'."""
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=dim ** -0.5 if scale is None else scale)
    if rot:
        m["rot"] = dict(base=base, dims=rot)
    if size is not None:
        m["mask"] = dict(size=size)
    if conv:
        m["conv"] = conv
    return m


def delta(heads, dim, gate_rank=8):
    return dict(heads=heads, dim=dim, gate_rank=gate_rank)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, groups=None, scale=None, shared=None):
    """``groups`` (count, keep). As a group's score is its best expert's, the groups only change a choice of more experts
    than groups are kept (top > keep)."""
    f = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if groups is not None:
        f["router"]["groups"] = dict(count=groups[0], keep=groups[1])
    if scale is not None:
        f["router"]["scale"] = scale
    if shared is not None:
        f["shared"] = dict(ff=shared)
    return f


def layer(kind, mixer, mlp=None):
    return dict(type=kind, mixer=mixer, mlp=mlp)


def config(layers, vocab=300, width=72, eps=1e-5, scale=3.0, mult=0.8, loop=None):
    c = dict(architecture="Tarupel", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale),
             residual_mult=mult, layers=layers)
    if loop is not None:
        c["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return c


def _mix():
    """Odd sizes everywhere, keys and values of different sizes, a stretch in the middle that runs three times."""
    return config([
        layer("attention", attention(6, 2, 20, 12, scale=0.3, rot=12, size=19, conv=3), dense(56)),
        layer("general_delta", delta(3, 12, gate_rank=5), moe(6, 3, 24, groups=(3, 2), scale=1.7, shared=40)),
        layer("attention_2", attention(4, 4, 16, 16, scale=0.4, rot=8, base=500.0, size=11), dense(40)),
        layer("general_delta", delta(2, 20), None),
        layer("attention_2", attention(6, 3, 12, 20, scale=0.4, rot=12, size=5), moe(4, 3, 16, scale=0.6)),
        layer("attention", attention(3, 3, 8, 8, rot=4, size=7, conv=5), moe(5, 1, 24, shared=16)),
    ], loop=(1, 3, 3))


def _wide():
    """Sizes that reach the tensor-core products and attention kernels; the loop starts at the first layer."""
    return config([
        layer("attention", attention(4, 2, 64, 64, scale=0.2, rot=32, base=1e6, size=50, conv=4), dense(136)),
        layer("general_delta", delta(4, 32, gate_rank=16), moe(8, 3, 64, groups=(4, 2), scale=2.0, shared=64)),
        layer("attention_2", attention(4, 1, 128, 128, scale=0.09, rot=128, size=70), moe(8, 4, 64, groups=(2, 1), shared=128)),
        layer("attention", attention(4, 4, 128, 128, scale=0.09, rot=64, size=90, conv=2), dense(128)),
    ], vocab=515, width=128, eps=1e-6, scale=8.0, mult=0.6, loop=(0, 2, 2))


def _one():
    """One of everything: one head, one tap, chunks and windows of one and two keys, one expert, a loop that runs once; no
    mask, no rotation, no convolution in some layers; factors of one."""
    return config([
        layer("attention", attention(1, 1, 8, 40, rot=8, size=1, conv=1), moe(1, 1, 16)),
        layer("attention_2", attention(3, 1, 8, 8, rot=2, size=1), None),
        layer("general_delta", delta(1, 8, gate_rank=1), dense(8)),
        layer("attention", attention(2, 1, 16, 8, size=2, conv=2), moe(3, 3, 8, groups=(3, 3), shared=8)),
        layer("attention", attention(2, 2, 8, 8, scale=1.0), None),
        layer("attention_2", attention(1, 1, 40, 8, size=2), moe(4, 1, 8, groups=(4, 1), scale=1.0)),
    ], width=40, scale=1.0, mult=1.0, loop=(2, 3, 1))


MIX, WIDE, ONE = _mix(), _wide(), _one()


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W = cfg["width"]
    shapes = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": ()}
    if cfg.get("loop"):
        shapes["loop.step"] = (cfg["loop"]["times"], W)
    for i, entry in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}.", entry["mixer"], entry["type"]
        shapes.update({p + "norm1": (), p + "ls1": (W,), p + "shift": (W,)})
        if kind == "general_delta":
            n, rank = m["heads"] * m["dim"], m["gate_rank"]
            for name in ("r", "k", "v", "g", "a"):
                shapes[p + "mix." + name] = (n, W)
            shapes.update({p + "mix.a.b": (n,), p + "mix.w1": (rank, W), p + "mix.w2": (n, rank), p + "mix.w0": (n,),
                           p + "mix.norm": (n,), p + "mix.o": (W, n)})
        else:
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for name, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                shapes.update({p + "mix." + name: (rows, W), p + f"mix.{name}.b": (rows,)})
                if kind == "attention" and m.get("conv"):
                    shapes[p + f"mix.{name}.conv"] = (rows, m["conv"])
            if kind == "attention_2":
                shapes.update({p + "mix.q.norm": (H * d,), p + "mix.k.norm": (G * d,)})
            shapes[p + "mix.o"] = (W, H * dv)
        f = entry.get("mlp")
        if f is None:
            continue
        shapes.update({p + "norm2": (), p + "ls2": (W,)})
        parts = [("", f["ff"])] if f["kind"] == "dense" else [(f"e{e}.", f["expert"]["ff"]) for e in range(f["router"]["experts"])]
        if f.get("shared"):
            parts.append(("shared.", f["shared"]["ff"]))
            shapes[p + "mlp.shared.sg"] = (1, W)
        for q, ff in parts:
            shapes.update({p + f"mlp.{q}gate": (ff, W), p + f"mlp.{q}up": (ff, W), p + f"mlp.{q}down": (W, ff)})
        if f["kind"] == "moe":
            shapes[p + "mlp.router"] = (f["router"]["experts"], W)
    return shapes


def draw_tensors(cfg: dict, seed: int, dtype=torch.float32) -> Dict[str, torch.Tensor]:
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=gen, dtype=torch.float32)
        leaf = name.split(".", 1)[1] if name.startswith("l") else name
        if leaf in ("norm1", "norm2", "ls1", "ls2", "mix.norm", "mix.q.norm", "mix.k.norm") or name == "final.norm":
            t = 1.0 + 0.2 * t
        elif leaf == "shift":
            t = 0.4 + 0.3 * t
        elif leaf.endswith(".b") or name in ("embed", "loop.step"):
            t = 0.5 * t
        elif leaf == "mix.w0":
            t = -2.0 + 1.5 * t
        elif leaf.endswith(".conv"):
            t = t / shape[-1] ** 0.5
        elif leaf == "mlp.router":
            t = 2.5 * t / shape[-1] ** 0.5
        elif leaf == "mlp.shared.sg":
            t = 2.0 * t / shape[-1] ** 0.5
        else:
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


def forward(cfg, w, tokens, residuals=None, choices=None) -> np.ndarray:
    return plain.Model(cfg, w, torch.float64).run(tokens, residuals=residuals, choices=choices).numpy()


def plain_logits(folder, requests) -> Dict[str, np.ndarray]:
    cfg, w = read_folder(folder)
    return {rid: forward(cfg, w, toks) for rid, toks in requests.items()}
