"""Shared by the Tatelorn tests: small configurations that differ in every size and option, model folders with random weights
in temporary places, and what the plain implementation (tests/plain_tatelorn.py) makes of them."""
from __future__ import annotations

import os
from typing import Dict, List

import torch

import plain_tatelorn as plain

F64 = torch.float64


def attention(heads, kv_heads, dim, vdim, scale, softcap=None, v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if softcap:
        m["softcap"] = softcap
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def layer(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def model(vocab, width, max_positions, eps, scale, logit_scale, layers):
    return {"architecture": "Tatelorn", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "logit_scale": logit_scale, "layers": layers}


# K: odd sizes everywhere; the first layer does not mix its values, the second is the first that does, one between the mixing ones
#    does not; values wider and narrower than keys (where no layer shares them the sizes differ too); 3:1, 2:1 and 1:1 grouping; a
#    layer without feed-forward; experts with and without a shared one; tight caps.
# L: sizes the bfloat16 fast products take; heads of 64, eight query heads on two; caps a bounded score cannot reach, reaches in part,
#    and none; a shared expert wider than the others, and one of their width.
# M: one head everywhere; no layer mixes; one expert, every expert chosen; factors below 1 and of 1.
# N: heads of 128 (the tcgen05 attention in bfloat16), four query heads on one, and eight on two; caps of both kinds; a dense layer
#    behind the routed ones.
# R: a width and sizes that are multiples of 4 only; values shared between layers whose keys differ in size.
CONFIGS = {
    "K": model(211, 96, 400, 1e-5, 3.7, 0.6, [
        layer(attention(6, 2, 24, 40, 0.3, 4.0, v_mix=False), dense(72)),
        layer(attention(6, 2, 16, 24, 0.35, 2.5), moe(5, 2, 48, 0.8, shared=(40, 1.3))),
        layer(attention(3, 3, 20, 12, 0.25, 9.0, v_mix=False), None),
        layer(attention(4, 2, 28, 24, 0.2, 30.0), moe(6, 3, 32, 2.0))]),
    "L": model(300, 128, 512, 1e-6, 11.3, 0.35, [
        layer(attention(8, 2, 64, 64, 0.125, 50.0), moe(8, 2, 64, 1.1, shared=(96, 0.9))),
        layer(attention(4, 2, 64, 64, 0.2, 14.0), dense(96)),
        layer(attention(8, 2, 64, 64, 0.15), moe(4, 1, 64, 0.7, shared=(64, 1.6)))]),
    "M": model(97, 64, 300, 1e-6, 1.0, 1.0, [
        layer(attention(1, 1, 8, 12, 0.5, 3.0, v_mix=False), moe(1, 1, 32, 0.5, shared=(16, 0.25))),
        layer(attention(1, 1, 32, 32, 0.2, v_mix=False), moe(3, 3, 16, 1.5))]),
    "N": model(331, 256, 640, 1e-6, 16.0, 0.5, [
        layer(attention(4, 1, 128, 128, 0.09, 40.0), moe(6, 2, 64, 1.4, shared=(64, 2.2))),
        layer(attention(8, 2, 128, 128, 0.088, 20.0, v_mix=False), None),
        layer(attention(6, 1, 128, 128, 0.1, 12.0), dense(160)),
        layer(attention(2, 1, 128, 128, 0.15, 6.0), moe(5, 2, 96, 0.9, shared=(128, 1.0)))]),
    "R": model(150, 100, 290, 1e-5, 0.5, 2.5, [
        layer(attention(5, 1, 20, 12, 0.3, 8.0), moe(3, 2, 36, 1.0, shared=(20, 0.6))),
        layer(attention(4, 1, 12, 12, 0.4, 5.0), dense(44)),
        layer(attention(3, 1, 44, 12, 0.2, 3.0), moe(4, 2, 20, 0.6, shared=(20, 0.6)))]),
}
BLOCK_SIZE = {"K": 16, "L": 8, "M": 32, "N": 16, "R": 16}
SEED = {"K": 61, "L": 62, "M": 63, "N": 64, "R": 65}


def write_case(tmp_path, name: str, store_dtype=torch.bfloat16, std: float = 0.1, config=None, steady: bool = False) -> str:
    """A model folder of configuration ``name`` with random weights.  ``std`` is large enough that attention weights and gates are far
    from uniform; the shares of the first layer's values are set apart (``set_shares``).  ``steady``: no router's choice is close
    (``steady_routers``)."""
    from iian_b200.config.registry import get_architecture
    from iian_b200.weights.random_init import write_model_folder
    from iian_b200.weights.safetensors_io import write_safetensors
    arch = get_architecture("Tatelorn")
    d = os.path.join(str(tmp_path), f"tatelorn{name}_{str(store_dtype).split('.')[-1]}" + ("_steady" if steady else ""))
    if not os.path.isdir(d):
        write_model_folder(d, arch, arch.load_config(config or CONFIGS[name]), seed=SEED.get(name, 1), store_dtype=store_dtype,
                           std=std, norm_jitter=0.4)
        path = os.path.join(d, "model.safetensors")
        w = plain.read_safetensors(path)
        set_shares(w)
        if steady:
            steady_routers(w)
        write_safetensors(path, {k: (v.to(store_dtype) if v.is_floating_point() else v) for k, v in w.items()}, metadata={"format": "pt"})
    return d


def set_shares(w: Dict[str, torch.Tensor]) -> None:
    """Shares of the first layer's values that no two layers have in common, one of them beyond 1/2, one negative."""
    for i, name in enumerate(sorted(k for k in w if k.endswith(".vmix"))):
        w[name] = torch.tensor([0.375, 0.6875, -0.25, 0.4375][i % 4])


def steady_routers(w: Dict[str, torch.Tensor], step: float = 1.5) -> None:
    """Random router weights put the logits of a few experts within a hair of each other for a good part of the tokens, and 16-bit
    rounding of the router's input then decides which expert a token takes: another expert is another output at full size.  So for
    the bfloat16 runs of whole models the stream's first column is made the same for every token (a constant in the tables, nothing
    added to it by the layers), and the routers read it with factors ``step`` apart, in a shuffled order that differs from layer to
    layer: no choice is close.  The weights stay the softmax the rest of the stream moves freely; the 32-bit runs and the kernels'
    own tests keep free choices."""
    w["pos"][:, 0] = 4.0
    w["embed"][:, 0] = 0.0
    # what stands in the column behind the embedding's norm depends a little on the rest of the row: about 4 / rms
    for k in list(w):
        if k.endswith(".norm1") or k.endswith(".norm2"):
            w[k][0] = -1.0
    for i, name in enumerate(sorted(k for k in w if k.endswith(".router"))):
        n = w[name].shape[0]
        order = torch.randperm(n, generator=torch.Generator().manual_seed(300 + i)).to(torch.float32)
        w[name][:, 0] = (order - (n - 1) / 2) * step


def plain_logits(model_dir: str, requests: Dict[str, List[int]]) -> Dict[str, torch.Tensor]:
    cfg, w = plain.load_folder(model_dir)
    return {rid: plain.forward(cfg, w, toks) for rid, toks in requests.items()}


def rounded_plain(folder, reqs, dtype: torch.dtype):
    """The plain implementation with the input and the result of every matrix product rounded to ``dtype``: how far rounding
    alone moves the logits at each position."""
    cfg, w = plain.load_folder(folder)
    plain.product_rounding = lambda z: z.to(dtype).to(F64)
    try:
        return {rid: plain.forward(cfg, w, toks) for rid, toks in reqs.items()}
    finally:
        plain.product_rounding = None


def owed(addend) -> torch.Tensor:
    """What a layer still has to add to the stream, in float64, worked out by hand from the addend it hands on."""
    y = addend.y.double()
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + addend.eps) * addend.weight.double()
