"""A plain, slow statement of the Tarupel decoder on the CPU, one function per mechanism, written from the design's
equations. It shares no code with the engine: tensors come in as a dict name -> torch tensor, the configuration as
the dict of config.json. A whole sequence runs at once, in one precision (float64 by default), without a cache: it is
the yardstick for prompts, decoding, portions and batches alike.

Notation: X [T, width] is the residual, H [T, width] a sublayer's input; W_x is the tensor '<layer>.mix.x' or
'<layer>.mlp.x', stored [out, in] and applied as W h.
"""
from __future__ import annotations

import math

import torch

UNIT_EPS = 1e-6
SUM_EPS = 1e-20


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def single_gain_norm(x, gain, eps):
    """The layers' norm: one number scales all coordinates."""
    return rms(x, eps) * gain


def shifted(H, mix):
    """Token shift: every coordinate moves from h_t towards h_(t-1) by the share ``mix`` (h_(-1) = 0)."""
    before = torch.cat([torch.zeros_like(H[:1]), H[:-1]])
    return H + (before - H) * mix


def rotated(x, base, dims, interleaved, positions=None):
    """x [T, heads, dim]: the pairs (i, i + dims / 2), or (2i, 2i + 1), of the first ``dims`` features turn by
    p * base^(-2i / dims)."""
    if not dims:
        return x
    p = torch.arange(x.shape[0], dtype=x.dtype) if positions is None else positions
    angle = p[:, None] * base ** (-2.0 * torch.arange(dims // 2, dtype=x.dtype) / dims)[None]
    c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
    y = x.clone()
    a, b = (slice(0, dims, 2), slice(1, dims, 2)) if interleaved else (slice(0, dims // 2), slice(dims // 2, dims))
    u, v = x[..., a], x[..., b]
    y[..., a], y[..., b] = u * c - v * s, v * c + u * s
    return y


def short_conv(U, weight):
    """Causal convolution per channel: y_t = sum_j weight[:, j] u_(t - taps + 1 + j), zeros before the start."""
    taps = weight.shape[1]
    padded = torch.cat([U.new_zeros(taps - 1, U.shape[1]), U])
    return sum(weight[:, j] * padded[j:j + U.shape[0]] for j in range(taps))


def window_mask(n, size):
    i = torch.arange(n)
    gap = i[:, None] - i[None, :]
    return (gap >= 0) & ((gap < size) if size else True)


def chunk_mask(n, size):
    i = torch.arange(n)
    seen = i[None, :] <= i[:, None]
    return seen & (i[:, None] // size == i[None, :] // size) if size else seen


def softmax_attention(q, k, v, scale, mask):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H * dv]; query head h reads key head h // (H / G)."""
    per = q.shape[1] // k.shape[1]
    out = []
    for h in range(q.shape[1]):
        score = (q[:, h] @ k[:, h // per].t()) * scale
        out.append(torch.softmax(score.masked_fill(~mask, -math.inf), dim=-1) @ v[:, h // per])
    return torch.cat(out, dim=-1)


def chunked_attention(w, m, eps, H):
    """Mixer 'attention': convolved q, k, v; half-split rotation, then q and k to unit root mean square per head;
    attention within chunks counted from the sequence's start."""
    def projected(name, size):
        y = H @ w[name].t() + w[name + ".b"]
        if name + ".conv" in w:
            y = short_conv(y, w[name + ".conv"])
        return y.view(H.shape[0], -1, size)
    rot = m.get("rot") or {}
    q, k = (rms(rotated(projected(n, m["dim"]), rot.get("base"), rot.get("dims", 0), False), eps) for n in ("q", "k"))
    return softmax_attention(q, k, projected("v", m["vdim"]), m["scale"],
                             chunk_mask(H.shape[0], (m.get("mask") or {}).get("size"))) @ w["o"].t()


def windowed_attention(w, m, eps, H):
    """Mixer 'attention_2': q and k normed over all their rows at once, interleaved rotation, a sliding window."""
    rot = m.get("rot") or {}

    def projected(name):
        return H @ w[name].t() + w[name + ".b"]
    q, k = (rotated((rms(projected(n), eps) * w[n + ".norm"]).view(H.shape[0], -1, m["dim"]), rot.get("base"),
                    rot.get("dims", 0), True) for n in ("q", "k"))
    return softmax_attention(q, k, projected("v").view(H.shape[0], -1, m["vdim"]), m["scale"],
                             window_mask(H.shape[0], (m.get("mask") or {}).get("size"))) @ w["o"].t()


def general_delta_rule(r, k, v, decay, rate, S):
    """S [heads, key, value]; r, k, decay, rate [T, heads, key]; v [T, heads, value]. Per head and token, with
    u = k / |k|:  S <- diag(decay) S - (rate u)(u^T S) + k v^T (both terms from the old S), o = S^T r."""
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + UNIT_EPS)
    out = []
    for t in range(r.shape[0]):
        along = torch.einsum("hk,hkv->hv", u[t], S)
        S = decay[t][:, :, None] * S - (rate[t] * u[t])[:, :, None] * along[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, r[t]))
    return torch.stack(out), S


def general_delta(w, m, eps, H):
    """Mixer 'general_delta'."""
    heads, d = m["heads"], m["dim"]

    def split(y):
        return y.view(H.shape[0], heads, d)
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(H @ w["w1"].t()) @ w["w2"].t() + w["w0"]))
    rate = torch.sigmoid(H @ w["a"].t() + w["a.b"])
    o, _ = general_delta_rule(*(split(H @ w[n].t()) for n in ("r", "k", "v")), split(decay), split(rate),
                              torch.zeros(heads, d, d, dtype=H.dtype))
    o = rms(o, eps).reshape(H.shape[0], heads * d) * w["norm"]
    return (o * torch.sigmoid(H @ w["g"].t())) @ w["o"].t()


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def dense(w, H):
    return (gelu_tanh(H @ w["gate"].t()) * (H @ w["up"].t())) @ w["down"].t()


def grouped_choice(scores, top, count, keep):
    """Indices of the ``top`` best scores among the experts of the ``keep`` groups (of ``count`` equal groups of
    neighbours) whose best scores are largest; scores [experts]."""
    if count > 1:
        groups = scores.view(count, -1)
        best = torch.topk(groups.max(dim=-1).values, keep).indices
        allowed = torch.zeros(count, dtype=torch.bool)
        allowed[best] = True
        scores = scores.masked_fill(~allowed.repeat_interleave(groups.shape[1]), -math.inf)
    return torch.topk(scores, top).indices


def gated_expert(w, prefix, h):
    return w[prefix + ".down"] @ (silu(w[prefix + ".gate"] @ h) * (w[prefix + ".up"] @ h))


def experts(w, f, H, choices=None):
    """Mixture of experts. ``choices``: if a list, receives every token's chosen experts."""
    r = f["router"]
    groups = r.get("groups") or {}
    out = []
    for h in H:
        s = torch.softmax(w["router"] @ h, dim=-1)
        chosen = grouped_choice(s, r["top"], groups.get("count", 1), groups.get("keep", 1))
        if choices is not None:
            choices.append(sorted(chosen.tolist()))
        weight = s[chosen] / (s[chosen].sum() + SUM_EPS) * r.get("scale", 1.0)
        y = sum(c * gated_expert(w, f"e{e}", h) for c, e in zip(weight, chosen.tolist()))
        if f.get("shared"):
            y = y + torch.sigmoid(w["shared.sg"] @ h) * gated_expert(w, "shared", h)
        out.append(y)
    return torch.stack(out)


MIXERS = {"attention": chunked_attention, "attention_2": windowed_attention, "general_delta": general_delta}


def run_order(cfg):
    """(layer, pass of the loop that starts here or None) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    body = [(i, t if i == start else None) for t in range(times) for i in range(start, stop)]
    return [(i, None) for i in range(start)] + body + [(i, None) for i in range(stop, n)]


class Model:
    def __init__(self, cfg, tensors, dtype=torch.float64):
        self.cfg = cfg
        self.w = {k: v.to(dtype) for k, v in tensors.items()}

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def run(self, tokens, residuals=None, choices=None):
        """Logits [T, vocab]. ``residuals``: if a list, receives the residual [T, width] after every layer run;
        ``choices``: if a list, the experts every token chose, layer run by layer run."""
        cfg, w = self.cfg, self.w
        eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
        first = w["embed"][torch.as_tensor(tokens)] * cfg.get("embedding", {}).get("scale", 1.0)
        X = first
        for i, loop_pass in run_order(cfg):
            if loop_pass is not None:
                if loop_pass > 0:
                    X = X + first
                X = X + w["loop.step"][loop_pass]
            layer, p = cfg["layers"][i], f"l{i}."
            H = shifted(single_gain_norm(X, w[p + "norm1"], eps), w[p + "shift"])
            X = X + m * (MIXERS[layer["type"]](self._sub(p + "mix."), layer["mixer"], eps, H) * w[p + "ls1"])
            f = layer.get("mlp")
            if f is not None:
                H, wf = single_gain_norm(X, w[p + "norm2"], eps), self._sub(p + "mlp.")
                y = dense(wf, H) if f["kind"] == "dense" else experts(wf, f, H, choices)
                X = X + m * (y * w[p + "ls2"])
            if residuals is not None:
                residuals.append(X)
        return single_gain_norm(X, w["final.norm"], eps) @ w["head"].t()
