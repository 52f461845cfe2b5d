"""An attention mixer whose heads are the difference of two softmax maps over the same values.

``q = Wq h`` (heads x 2 x dim), ``k = Wk h`` (kv_heads x 2 x dim), ``v = Wv h`` (kv_heads x v_dim), no biases; a head's two maps
lie side by side.  The first ``rot`` entries of every map of q and k are rotated by the position (entry 2i with entry 2i + 1; the
part in ``position`` gives the frequencies, possibly rescaled for long contexts, and a magnitude on cos and sin).  Head ``g``
reads KV head ``g // (heads / kv_heads)``; per map

    s_ij = (q_i . k_j) * scale,    s <- cap tanh(s / cap)  (``softcap``),    key j visible to position i  iff  j <= i

and a softmax over the visible keys.  With ``a1`` and ``a2`` the two maps' weighted sums of the SAME values and one number per
layer ``lam = exp(lq1 . lk1) - exp(lq2 . lk2) + diff``,

    o = a1 - lam a2,    o <- o / sqrt(mean(o^2) + eps) * (1 - diff)    (over the head's v_dim values)

and ``Wo`` on the concatenated heads.

``Wq | Wk | Wv`` are one product.  The cache is a K/V page cache whose key cells hold both maps (2 x dim entries) and whose value
cells have ``v_dim`` entries: a value is stored and fetched once for both maps.
"""
from __future__ import annotations

import math
from typing import Dict

import torch

from .. import ops
from ..config.spec import PartSpec
from ..weights.loader import TensorSpec
from .base import KVNeed, Mixer, POSITIONS, register_mixer

MAX_DIM = 512                   # what the general kernel holds per map and per value


@register_mixer("difference_attention")
class DifferenceAttention(Mixer):
    """params: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim`` (of one map), ``v_dim``, ``scale``, ``softcap`` (None:
    scores as they are), ``diff``, ``norm_eps``, ``position`` (a PartSpec: ``rotary`` or ``scaled_rotary`` in the interleaved style,
    or ``none``)."""

    def __init__(self, spec, dtype, device):
        super().__init__(spec, dtype, device)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.nh = int(p["num_heads"])
        self.nkv = int(p["num_kv_heads"])
        self.hd = int(p["head_dim"])
        self.vd = int(p["v_dim"])
        if self.nkv <= 0 or self.nh % self.nkv:
            raise ValueError(f"difference_attention: {self.nh} heads cannot share {self.nkv} KV heads")
        if max(self.hd, self.vd) > MAX_DIM:
            raise ValueError(f"difference_attention: maps and values of up to {MAX_DIM} entries")
        self.scale = float(p["scale"])
        cap = p.get("softcap")
        self.softcap = float(cap) if cap else None
        if self.softcap is not None and self.softcap <= 0:
            raise ValueError("difference_attention: softcap must be positive or None")
        self.diff = float(p["diff"])
        self.eps = float(p["norm_eps"])
        self.position = POSITIONS.build(p.get("position") or PartSpec("none"), dtype, device)
        self.rot = int(getattr(self.position, "dim", 0) or 0)
        if self.rot > self.hd:
            raise ValueError(f"difference_attention: the position encoding rotates {self.rot} entries of a map of {self.hd}")
        if self.rot and getattr(self.position, "style", 1) != 1:
            raise ValueError("difference_attention: pairs are (2i, 2i + 1)")
        self.q_size = self.nh * 2 * self.hd
        self.k_size = self.nkv * 2 * self.hd
        self.v_size = self.nkv * self.vd
        self.w_in = self.w_o = None
        self.lam = 0.0

    def tensors(self) -> Dict[str, TensorSpec]:
        t = {"q": TensorSpec((self.q_size, self.hidden)), "k": TensorSpec((self.k_size, self.hidden)),
             "v": TensorSpec((self.v_size, self.hidden)), "o": TensorSpec((self.hidden, self.nh * self.vd))}
        for n in ("lq1", "lk1", "lq2", "lk2"):
            t[n] = TensorSpec((self.hd,), init="zeros_jitter")
        return t

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        ws = [tensors["q"], tensors["k"], tensors["v"]]
        if len({w.dtype for w in ws}) > 1:
            ws = [w.to(torch.float32) for w in ws]
        self.w_in = torch.cat(ws, dim=0).contiguous()            # columns of the product: q | k | v
        self.w_o = tensors["o"].contiguous()
        dot = [float((tensors[f"lq{m}"].double() * tensors[f"lk{m}"].double()).sum()) for m in (1, 2)]
        self.lam = math.exp(dot[0]) - math.exp(dot[1]) + self.diff

    def cache_need(self) -> KVNeed:
        return KVNeed(self.nkv, 2 * self.hd, None, self.vd if self.vd != 2 * self.hd else None)

    def _fast(self) -> bool:
        return self.dtype == torch.bfloat16 and self.hd == 64 and self.vd == 128 and self.scale > 0

    def kernel_libraries(self):
        return ("difference_attention", "gemm_simt") + (("window_attention",) if self.rot else ()) \
            + (("difference_attention_mma", "attention_tc") if self._fast() else ())

    def graph_plan(self, num_seqs: int, max_ctx: int):
        k = ops.kernels()
        if not hasattr(k, "difference_attention_plan"):
            return None
        return k.difference_attention_plan(num_seqs, self.nkv, self.hd, self.vd, self.scale, max_ctx, self.dtype)

    def forward(self, x, ctx, cache, writes_cache: bool):
        if not writes_cache:
            raise ValueError("difference_attention: a layer of this kind fills its own cache")
        k = ops.kernels()
        n = x.shape[0]
        proj = ctx.buf("difference_in", (n, self.w_in.shape[0]), self.dtype)
        k.linear(x, self.w_in, proj)
        meta = ctx.page_meta(cache.group)
        table = self.position.table64(ctx) if self.rot else None
        q = ctx.buf("q", (n, self.q_size), self.dtype)
        k.rotate_pairs_store(proj, 0, self.q_size, self.q_size + self.k_size, q, cache.k, cache.v, table, meta.slots,
                             num_heads=2 * self.nh, num_kv_heads=self.nkv, maps=2, k_dim=self.hd, v_dim=self.vd, rot_dim=self.rot)
        plan = ctx.graph_plan(self)
        attn = ctx.buf("attn", (n, self.nh * self.vd), self.dtype)
        k.difference_attention(q, cache.k, cache.v, attn, meta, num_heads=self.nh, num_kv_heads=self.nkv, k_dim=self.hd,
                               v_dim=self.vd, scale=self.scale, softcap=self.softcap, lam=self.lam, factor=1.0 - self.diff,
                               eps=self.eps, **({"n_split": plan["n_split"]} if plan else {}))
        out = ctx.buf("mixer_out", (n, self.hidden), self.dtype)
        k.linear(attn, self.w_o, out)
        return out
