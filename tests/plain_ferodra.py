"""A plain, slow implementation of the Ferodra design: whole sequences, no cache, one function per mechanism.

It shares no code with ``iian_b200``: it takes a configuration (the ``config.json`` mapping) and the tensors by their
file names and computes with elementary torch operations on the CPU, in float64 by default, so that it can serve as the
oracle of the 32-bit and of the bfloat16 path.

Notation.  ``x`` [T, W] is the stream of one sequence, positions ``0 .. T-1``.  A layer has a norm before AND after each
sub-layer and a factor per column behind the second:

    x' = x + c1 * n1b(mixer(n1(x)));    x'' = x' + c2 * n2b(ff(n2(x')))

with ``n(y) = w tanh(a y) + b`` (no statistics of the row).  A stretch of layers may run several times in a row with the
same weights; run ``t`` starts with ``x <- x + step_t``.  The recurrent mixer is walked token by token and can be given a
state to start from and asked for the state it ends with, so that a test can cut a sequence anywhere.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Mapping, Optional

import torch

from plain_qwen3 import read_safetensors


def load_folder(model_dir: str):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))


# ---- elementary pieces ------------------------------------------------------------------------------
product_rounding = None         # a rounding applied around every matrix product, for tests of rounding sensitivity


def mm(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    if product_rounding is None:
        return h @ w.T
    return product_rounding(product_rounding(h) @ w.T)


def tanh_norm(x: torch.Tensor, w: Mapping[str, torch.Tensor], name: str) -> torch.Tensor:
    """``tanh(a x) w + b`` with one number ``a`` for the whole norm."""
    return torch.tanh(w[name + ".alpha"].reshape(()) * x) * w[name] + w[name + ".b"]


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def over_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_length(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


# ---- rotation ---------------------------------------------------------------------------------------
def rotation(rot: Optional[Mapping]):
    """``(frequencies float64, factor on cos and sin)``; without ``scaling`` the plain ones."""
    if rot is None:
        return torch.zeros(0, dtype=torch.float64), 1.0
    n, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if sc is None:
        return torch.tensor(f, dtype=torch.float64), 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def where(turns: float) -> float:
        return n * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(where(float(sc["fast"]))), 0)
    hi = min(math.ceil(where(float(sc["slow"]))), n - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def rotate_neighbours(v: torch.Tensor, pos: torch.Tensor, freqs: torch.Tensor, factor: float) -> torch.Tensor:
    """Entries 2i and 2i+1 of the last axis turn by ``pos * freqs[i]``; entries behind the last pair pass unchanged.
    ``v``: [T, heads, n]."""
    out = v.clone()
    for i in range(freqs.numel()):
        ang = pos.to(torch.float64) * freqs[i]
        c = (torch.cos(ang) * factor).to(v.dtype)[:, None]
        s = (torch.sin(ang) * factor).to(v.dtype)[:, None]
        out[..., 2 * i] = v[..., 2 * i] * c - v[..., 2 * i + 1] * s
        out[..., 2 * i + 1] = v[..., 2 * i + 1] * c + v[..., 2 * i] * s
    return out


# ---- attention with the difference of two softmax maps ---------------------------------------------------
def capped_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, cap: Optional[float], q_pos0: int = 0) -> torch.Tensor:
    """One map of one head: ``q`` [Tq, d] at positions ``q_pos0 ..``, ``k`` [Tk, d], ``v`` [Tk, dv] at ``0 ..``; causal."""
    s = (q @ k.T) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    i = q_pos0 + torch.arange(q.shape[0])[:, None]
    s = s.masked_fill(torch.arange(k.shape[0])[None, :] > i, -math.inf)
    p = torch.exp(s - s.max(-1, keepdim=True).values)
    return (p / p.sum(-1, keepdim=True)) @ v


def map_weight(w: Mapping[str, torch.Tensor], pre: str, diff: float) -> torch.Tensor:
    """What the second map is multiplied by, one number per layer."""
    return torch.exp((w[pre + "lq1"] * w[pre + "lk1"]).sum()) - torch.exp((w[pre + "lq2"] * w[pre + "lk2"]).sum()) + diff


def map_difference(q, k, v, scale: float, cap: Optional[float], lam, diff: float, eps: float, q_pos0: int = 0) -> torch.Tensor:
    """``q`` [Tq, H, 2, d], ``k`` [Tk, G, 2, d], ``v`` [Tk, G, dv] -> [Tq, H, dv]: map 1 minus ``lam`` times map 2, divided by
    its root mean square per head, times ``1 - diff``."""
    H, G = q.shape[1], k.shape[1]
    out = torch.zeros(q.shape[0], H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        a = [capped_attention(q[:, h, m], k[:, g, m], v[:, g], scale, cap, q_pos0) for m in (0, 1)]
        out[:, h] = over_rms(a[0] - lam * a[1], eps) * (1.0 - diff)
    return out


def attention_mixer(cfg: Mapping, w: Mapping[str, torch.Tensor], pre: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = int(cfg["heads"]), int(cfg["kv_heads"]), int(cfg["dim"]), int(cfg["vdim"])
    freqs, factor = rotation(cfg.get("rot"))
    pos = torch.arange(T)
    q = rotate_neighbours(mm(h, w[pre + "q"]).view(T, H * 2, d), pos, freqs, factor).view(T, H, 2, d)
    k = rotate_neighbours(mm(h, w[pre + "k"]).view(T, G * 2, d), pos, freqs, factor).view(T, G, 2, d)
    v = mm(h, w[pre + "v"]).view(T, G, dv)
    diff = float(cfg["diff"])
    cap = cfg.get("softcap")
    o = map_difference(q, k, v, float(cfg["scale"]), float(cap) if cap else None, map_weight(w, pre, diff), diff, eps)
    return mm(o.reshape(T, H * dv), w[pre + "o"])


# ---- the delta rule with one decay per head ---------------------------------------------------------------
def short_convolution(x: torch.Tensor, taps: torch.Tensor, before: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``y_t[c] = sum_j taps[c, j] x_{t - (n - 1) + j}[c]``; ``before``: the ``n - 1`` rows ahead of ``x`` (None: zeros)."""
    n = taps.shape[1]
    if before is None:
        before = torch.zeros(n - 1, x.shape[1], dtype=x.dtype)
    ext = torch.cat([before, x], dim=0)
    y = torch.zeros_like(x)
    for j in range(n):
        y = y + taps[:, j] * ext[j: j + x.shape[0]]
    return y


def delta_scan(q, k, v, beta, g, state=None):
    """``q``, ``k`` [T, H, d], ``v`` [T, H, dv], ``beta``, ``g`` [T, H].  Per token ``S <- g S; u = beta (v - S^T k);
    S <- S + k u^T; o = S^T q``.  Returns ``(o, S)``, ``S`` [H, d, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    o = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o, S


def delta_mixer(cfg: Mapping, w: Mapping[str, torch.Tensor], pre: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = int(cfg["heads"]), int(cfg["kv_heads"]), int(cfg["dim"]), int(cfg["vdim"])
    q = silu(short_convolution(mm(h, w[pre + "q"]), w[pre + "q.conv"])).view(T, G, d)
    k = silu(short_convolution(mm(h, w[pre + "k"]), w[pre + "k.conv"])).view(T, G, d)
    v = silu(short_convolution(mm(h, w[pre + "v"]), w[pre + "v.conv"])).view(T, H, dv)
    q, k = unit_length(q) * d ** -0.5, unit_length(k)
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(mm(h, w[pre + "b"]))
    g = torch.exp(-torch.exp(w[pre + "A_log"]) * torch.nn.functional.softplus(mm(h, w[pre + "a"]) + w[pre + "dt_bias"]))
    o, _ = delta_scan(q, k, v, beta, g)
    y = over_rms(o, eps) * w[pre + "norm"]
    return mm(y.reshape(T, H * dv) * silu(mm(h, w[pre + "g"])), w[pre + "o"])


# ---- feed-forward -----------------------------------------------------------------------------------
def gated_feed_forward(h: torch.Tensor, w: Mapping[str, torch.Tensor], pre: str) -> torch.Tensor:
    return mm(silu(mm(h, w[pre + "gate"])) * mm(h, w[pre + "up"]), w[pre + "down"])


def squared_relu_expert(h: torch.Tensor, w: Mapping[str, torch.Tensor], pre: str) -> torch.Tensor:
    return mm(torch.relu(mm(h, w[pre + "up"])) ** 2, w[pre + "down"])


# A test that wants to know where a router's choice hangs on a hair sets this to a list; every call then appends, per token,
# the gap between the last chosen choice score and the best one left out (infinity where everything is chosen).
router_margins: Optional[list] = None


def router_choice(h: torch.Tensor, w: Mapping[str, torch.Tensor], pre: str, top: int, scale: float):
    """``(ids [T, top], weights [T, top])``: the largest of softmax + correction; the weights are the softmax alone, scaled."""
    s = torch.softmax(h @ w[pre + "router"].T, dim=-1)
    choice = s + w[pre + "correction"]
    ids = torch.sort(choice, dim=-1, descending=True, stable=True).indices
    if router_margins is not None:
        left = torch.gather(choice, 1, ids[:, top: top + 1])[:, 0] if top < s.shape[-1] else torch.full_like(s[:, 0], -math.inf)
        router_margins.append(torch.gather(choice, 1, ids[:, top - 1: top])[:, 0] - left)
    ids = ids[:, :top]
    return ids, torch.gather(s, 1, ids) * scale


def experts_feed_forward(cfg: Mapping, w: Mapping[str, torch.Tensor], pre: str, h: torch.Tensor) -> torch.Tensor:
    r = cfg["router"]
    ids, wts = router_choice(h, w, pre, int(r["top"]), float(r.get("scale", 1.0)))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for c in range(ids.shape[1]):
            e = int(ids[t, c])
            y = squared_relu_expert(h[t: t + 1], w, f"{pre}e{e}.")[0] if e < int(r["experts"]) else h[t]      # else: identity
            out[t] += wts[t, c] * y
    if cfg.get("shared") is not None:
        out = out + torch.sigmoid(mm(h, w[pre + "shared.sg"])) * squared_relu_expert(h, w, pre + "shared.")
    return out


# ---- the model --------------------------------------------------------------------------------------
def run_order(cfg: Mapping) -> List[tuple]:
    """(layer, number of the run of the repeated stretch that starts here, or None)."""
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if lp is None:
        return [(i, None) for i in range(n)]
    start, stop, times = int(lp["start"]), int(lp["stop"]), int(lp["times"])
    order = [(i, None) for i in range(start)]
    for t in range(times):
        order += [(i, t if i == start else None) for i in range(start, stop)]
    return order + [(i, None) for i in range(stop, n)]


def forward(cfg: Mapping, weights: Mapping[str, torch.Tensor], tokens, dtype=torch.float64, return_layers: bool = False):
    """Logits [T, vocab] of one sequence (and, if asked, the stream after every layer run)."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)].clone()
    streams = []
    for i, t in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = x + w["loop.step"][t]
        mixer = {"attention": attention_mixer, "delta": delta_mixer}[layer["type"]]
        y = mixer(layer["mixer"], w, p + "mix.", tanh_norm(x, w, p + "norm1"), eps)
        x = x + tanh_norm(y, w, p + "norm1b") * w[p + "ls1"]
        if layer.get("mlp") is not None:
            h = tanh_norm(x, w, p + "norm2")
            y = gated_feed_forward(h, w, p + "mlp.") if layer["mlp"]["kind"] == "dense" else experts_feed_forward(layer["mlp"], w, p + "mlp.", h)
            x = x + tanh_norm(y, w, p + "norm2b") * w[p + "ls2"]
        streams.append(x.clone())
    logits = tanh_norm(x, w, "final.norm") @ w["embed"].T
    return (logits, torch.stack(streams)) if return_layers else logits
