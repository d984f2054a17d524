"""A plain, slow statement of the Zetonex decoder on the CPU, one function per mechanism, written from the design's
equations. It shares no code with the engine: tensors come in as a dict name -> torch tensor, the configuration as
the dict of config.json. A whole sequence runs at once, in one precision (float64 by default), without a cache: it is
the yardstick for prompts, decoding, portions and batches alike.

Notation: X [T, width] is the residual, H [T, width] what a layer's sublayers read; W_x is the tensor '<layer>.mix.x' or
'<layer>.mlp.x', stored [out, in] and applied as W h.
"""
from __future__ import annotations

import math

import torch

GLU_ALPHA = 1.702


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """The layers' norm: a weight stored around zero."""
    return rms(x, eps) * (1.0 + w)


def frequencies(rot, dtype=torch.float64):
    """Turns per position of every pair, with long wavelengths slowed down where ``rot['scaling']`` asks for it."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            length = 2.0 * math.pi / f
            if length > s["original"] / s["low"]:
                f = f / s["factor"]
            elif length >= s["original"] / s["high"]:
                share = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - share) * f / s["factor"] + share * f
        out.append(f)
    return torch.tensor(out, dtype=dtype)


def rotated(x, rot):
    """x [T, heads, dim]: the pairs (i, i + dims / 2) of the first ``dims`` features turn by position * frequency."""
    if not rot or not rot.get("dims"):
        return x
    half = rot["dims"] // 2
    angle = torch.arange(x.shape[0], dtype=x.dtype)[:, None] * frequencies(rot, x.dtype)[None]
    c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


def seen(n, size, keep_first=0):
    """[n, n] mask: position i sees j <= i if j is among the last ``size`` positions (None: all) or the first ``keep_first``."""
    i = torch.arange(n)
    gap = i[:, None] - i[None, :]
    near = torch.ones(n, n, dtype=torch.bool) if size is None else gap < size
    return (gap >= 0) & (near | (i[None, :] < keep_first))


def softmax_weights(q, k, scale, mask, softcap=None):
    """[T, T] attention weights of one query head's rows q [T, d] over one key head's rows k [T, d]."""
    score = (q @ k.t()) * scale
    if softcap is not None:
        score = softcap * torch.tanh(score / softcap)
    return torch.softmax(score.masked_fill(~mask, -math.inf), dim=-1)


def gated_attention(w, m, eps, H):
    """Mixer 'attention': the values are the keys before their rotation; a window with kept first tokens; a sigmoid gate on
    every feature of the heads side by side."""
    T, heads, groups, d = H.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (H @ w["q"].t()).view(T, heads, d)
    v = (H @ w["k"].t()).view(T, groups, d)
    q, k = rotated(q, m.get("rot")), rotated(v, m.get("rot"))
    mask = seen(T, (m.get("mask") or {}).get("size"), (m.get("mask") or {}).get("keep_first", 0))
    out = [softmax_weights(q[:, h], k[:, h * groups // heads], m["scale"], mask) @ v[:, h * groups // heads]
           for h in range(heads)]
    return (torch.cat(out, dim=-1) * torch.sigmoid(H @ w["g"].t())) @ w["o"].t()


def difference_share(w, diff):
    """lambda, one number a layer."""
    return (torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff).item()


def differential_attention(w, m, eps, H):
    """Mixer 'attention_2': two attention maps a head over the same values, the second one's output subtracted."""
    T, heads, groups, d, dv = H.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotated(rms((H @ w["q"].t()).view(T, heads * 2, d), eps) * w["q.norm"], m.get("rot")).view(T, heads, 2, d)
    k = rotated(rms((H @ w["k"].t()).view(T, groups * 2, d), eps) * w["k.norm"], m.get("rot")).view(T, groups, 2, d)
    v = (H @ w["v"].t()).view(T, groups, dv)
    mask = seen(T, (m.get("mask") or {}).get("size"))
    share = difference_share(w, m["diff"])
    out = []
    for h in range(heads):
        g = h * groups // heads
        a1, a2 = (softmax_weights(q[:, h, i], k[:, g, i], m["scale"], mask, m.get("softcap")) @ v[:, g] for i in (0, 1))
        out.append(rms(a1 - share * a2, eps) * (1.0 - m["diff"]))
    return torch.cat(out, dim=-1) @ w["o"].t()


def dense(w, H):
    z = H @ w["gate"].t() + w["gate.b"]
    return (z * torch.sigmoid(z) * (H @ w["up"].t() + w["up.b"])) @ w["down"].t() + w["down.b"]


def clamped_expert(w, prefix, h, limit):
    g = torch.clamp(w[prefix + ".gate"] @ h, max=limit)
    u = torch.clamp(w[prefix + ".up"] @ h, min=-limit, max=limit)
    return w[prefix + ".down"] @ (g * torch.sigmoid(GLU_ALPHA * g) * (u + 1.0))


def table_experts(w, f, H, tokens):
    """Mixture of experts without a router: a row of the table names the experts of a token id, all of one weight."""
    top = f["router"]["top"]
    return torch.stack([sum(clamped_expert(w, f"e{e}", h, f["expert"]["limit"]) for e in w["table"][t].long().tolist()) / top
                        for h, t in zip(H, tokens)])


MIXERS = {"attention": gated_attention, "attention_2": differential_attention}


def run_order(cfg):
    """(layer, True where a pass of the loop starts) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    body = [(i, i == start) for i in range(start, stop)] * times
    return [(i, False) for i in range(start)] + body + [(i, False) for i in range(stop, n)]


class Model:
    def __init__(self, cfg, tensors, dtype=torch.float64):
        self.cfg = cfg
        self.w = {k: v.to(dtype) for k, v in tensors.items()}

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def run(self, tokens, residuals=None):
        """Logits [T, vocab]. ``residuals``: if a list, receives the residual [T, width] after every layer run."""
        cfg, w = self.cfg, self.w
        eps = cfg["norm"]["eps"]
        tokens = [int(t) for t in tokens]
        first = w["embed"][torch.as_tensor(tokens)]
        X = first
        for i, starts_pass in run_order(cfg):
            if starts_pass:
                X = torch.cat([X, first], dim=-1) @ w["loop.in"].t()
            layer, p = cfg["layers"][i], f"l{i}."
            H = centred_norm(X, w[p + "norm1"], eps)
            y = MIXERS[layer["type"]](self._sub(p + "mix."), layer["mixer"], eps, H)
            f = layer.get("mlp")
            if f is not None:
                wf = self._sub(p + "mlp.")
                y = y + (dense(wf, H) if f["kind"] == "dense" else table_experts(wf, f, H, tokens))
            X = X + y
            if residuals is not None:
                residuals.append(X)
        return centred_norm(X, w["final.norm"], eps) @ w["head"].t() * cfg.get("logit_scale", 1.0)
