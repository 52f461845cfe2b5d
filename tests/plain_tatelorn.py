"""A plain, slow implementation of the Tatelorn design: whole sequences, no cache, one function per mechanism.

It shares no code with ``iian_b200``: it takes a configuration (the ``config.json`` mapping) and the tensors by their
file names and computes with elementary torch operations on the CPU, in float64 by default, so that it can serve as the
oracle of the 32-bit and of the bfloat16 path.

Notation.  ``x`` [T, W] is the stream of one sequence, positions ``0 .. T-1``.  It starts as ``n_e(a E[token] + P[position])``;
a layer normalises what it ADDS and reads the stream as it is:

    x' = x + n1(mixer(x));    x'' = x' + n2(ff(x'))

with ``n(y) = y / sqrt(mean(y^2) + eps) (1 + w)``; at the end ``logits = b E n_f(x)``.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, Mapping, Optional

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


def over_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """The model's norm: the stored weight sits around zero."""
    return over_rms(x, eps) * (1.0 + weight)


def placed_embedding(w: Mapping[str, torch.Tensor], tokens, scale: float, eps: float) -> torch.Tensor:
    """The token's row times ``scale`` plus the position's own row, normalised."""
    ids = torch.as_tensor(tokens, dtype=torch.long)
    return centred_norm(w["embed"][ids] * scale + w["pos"][: ids.numel()], w["embed.norm"], eps)


# ---- attention --------------------------------------------------------------------------------------
def capped_softmax_head(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, cap: Optional[float],
                        q_pos0: int = 0) -> torch.Tensor:
    """One head: ``q`` [Tq, d] at positions ``q_pos0 ..``, ``k`` [Tk, d], ``v`` [Tk, dv] at ``0 ..``; causal; scores through
    the cap; the denominator holds one more than the visible keys' exponentials."""
    s = (q @ k.T) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    i = q_pos0 + torch.arange(q.shape[0])[:, None]
    seen = torch.arange(k.shape[0])[None, :] <= i
    m = s.masked_fill(~seen, 0.0).max(-1, keepdim=True).values.clamp(min=0.0)        # at least the extra term's own score, 0
    p = torch.exp(s - m) * seen
    return (p / (torch.exp(-m) + p.sum(-1, keepdim=True))) @ v


def grouped_attention(q, k, v, scale: float, cap: Optional[float], q_pos0: int = 0) -> torch.Tensor:
    """``q`` [Tq, H, d], ``k`` [Tk, G, d], ``v`` [Tk, G, dv] -> [Tq, H, dv]."""
    H, G = q.shape[1], k.shape[1]
    out = torch.zeros(q.shape[0], H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        out[:, h] = capped_softmax_head(q[:, h], k[:, g], v[:, g], scale, cap, q_pos0)
    return out


def mixed_values(v: torch.Tensor, first: Optional[torch.Tensor], share) -> torch.Tensor:
    """The layer's values with a share of the first mixing layer's values of the same tokens (None: this is the first)."""
    return v if first is None else (1.0 - share) * v + share * first


def attention_mixer(cfg: Mapping, w: Mapping[str, torch.Tensor], pre: str, h: torch.Tensor, eps: float, first: Optional[torch.Tensor]):
    """``(output, the values as this layer uses them)``."""
    T = h.shape[0]
    H, G, d, dv = int(cfg["heads"]), int(cfg["kv_heads"]), int(cfg["dim"]), int(cfg["vdim"])
    q = over_rms(mm(h, w[pre + "q"]).view(T, H, d), eps) * w[pre + "q.norm"]
    k = over_rms(mm(h, w[pre + "k"]).view(T, G, d), eps) * w[pre + "k.norm"]
    v = mm(h, w[pre + "v"]).view(T, G, dv)
    if cfg.get("v_mix") and first is not None:
        v = mixed_values(v, first, w[pre + "vmix"].reshape(()))
    cap = cfg.get("softcap")
    o = grouped_attention(q, k, v, float(cfg["scale"]), float(cap) if cap else None)
    return mm(o.reshape(T, H * dv), w[pre + "o"]), v


# ---- feed-forward -----------------------------------------------------------------------------------
def relu_feed_forward(h: torch.Tensor, w: Mapping[str, torch.Tensor], pre: str) -> torch.Tensor:
    return mm(torch.relu(mm(h, w[pre + "gate"])) * mm(h, w[pre + "up"]), w[pre + "down"])


def clipped_expert(h: torch.Tensor, w: Mapping[str, torch.Tensor], pre: str, limit: float) -> torch.Tensor:
    g = mm(h, w[pre + "gate"]).clamp(max=limit)
    u = mm(h, w[pre + "up"]).clamp(min=-limit, max=limit)
    return mm(g * torch.sigmoid(1.702 * g) * (u + 1.0), w[pre + "down"])


# A test that wants to know where a router's choice hangs on a hair sets this to a list; every call then appends, per token,
# the gap between the last chosen logit and the best one left out (infinity where everything is chosen).
router_margins: Optional[list] = None


def router_choice(h: torch.Tensor, w: Mapping[str, torch.Tensor], pre: str, top: int):
    """``(ids [T, top], weights [T, top])``: the largest logits; the weights are the softmax over the chosen ones."""
    z = h @ w[pre + "router"].T
    ids = torch.sort(z, dim=-1, descending=True, stable=True).indices
    if router_margins is not None:
        left = torch.gather(z, 1, ids[:, top: top + 1])[:, 0] if top < z.shape[-1] else torch.full_like(z[:, 0], -math.inf)
        router_margins.append(torch.gather(z, 1, ids[:, top - 1: top])[:, 0] - left)
    ids = ids[:, :top]
    return ids, torch.softmax(torch.gather(z, 1, ids), dim=-1)


def experts_feed_forward(cfg: Mapping, w: Mapping[str, torch.Tensor], pre: str, h: torch.Tensor) -> torch.Tensor:
    ids, wts = router_choice(h, w, pre, int(cfg["router"]["top"]))
    limit = float(cfg["expert"]["limit"])
    out = torch.zeros_like(h)
    for e in range(int(cfg["router"]["experts"])):
        rows, choice = torch.nonzero(ids == e, as_tuple=True)
        if rows.numel():
            out[rows] += wts[rows, choice][:, None] * clipped_expert(h[rows], w, f"{pre}e{e}.", limit)
    if cfg.get("shared") is not None:
        out = out + torch.sigmoid(mm(h, w[pre + "shared.sg"])) * clipped_expert(h, w, pre + "shared.", float(cfg["shared"]["limit"]))
    return out


# ---- the model --------------------------------------------------------------------------------------
def forward(cfg: Mapping, weights: Mapping[str, torch.Tensor], tokens, dtype=torch.float64, return_layers: bool = False):
    """Logits [T, vocab] of one sequence (and, if asked, the stream after every layer)."""
    w: Dict[str, torch.Tensor] = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = placed_embedding(w, tokens, float(cfg["embedding"]["scale"]), eps)
    streams, first = [], None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y, v = attention_mixer(layer["mixer"], w, p + "mix.", x, eps, first)
        if layer["mixer"].get("v_mix") and first is None:
            first = v
        x = x + centred_norm(y, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            y = relu_feed_forward(x, w, p + "mlp.") if layer["mlp"]["kind"] == "dense" else experts_feed_forward(layer["mlp"], w, p + "mlp.", x)
            x = x + centred_norm(y, w[p + "norm2"], eps)
        streams.append(x.clone())
    logits = centred_norm(x, w["final.norm"], eps) @ w["embed"].T * float(cfg["logit_scale"])
    return (logits, torch.stack(streams)) if return_layers else logits
