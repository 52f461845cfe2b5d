"""Shared by the Ferodra tests: small configurations that differ in every size and option, model folders with random weights
in temporary places, and what the plain implementation (tests/plain_ferodra.py) makes of them."""
from __future__ import annotations

import os
from typing import Dict, List

import torch

import plain_ferodra as plain

F64 = torch.float64


def rot(dims, base, **scaling):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = scaling
    return r


def attention(heads, kv_heads, dim, vdim, scale, diff, softcap=None, rotation=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if softcap:
        m["softcap"] = softcap
    if rotation:
        m["rot"] = rotation
    return {"type": "attention", "mixer": m}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff, scale, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "scale": scale}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def layer(mix, mlp):
    return dict(mix, mlp=mlp)


# K: odd sizes everywhere; the repeated stretch starts behind the first layer and is followed by another; values wider and
#    narrower than keys; partial rotation with a ramp that begins and ends inside the pairs; 3:1, 2:1 and 1:1 grouping; a layer
#    without feed-forward; experts with and without a shared one, one identity output and three; a tight cap.
# L: sizes the bfloat16 fast products take (multiples of 32); the first two layers run three times; maps of 64 over values of
#    128 (the tensor-core attention in bfloat16), eight query heads on two; a recurrence wider than it is deep.
# M: no repetition; one head everywhere; no rotation, no cap, a plain rotation (no rescaling); one tap (no convolution state);
#    every router output chosen; no identity output; a recurrence deep enough for many entries a lane.
# N: maps of 64 over values of 128 with four query heads on one; a recurrence of 128 x 128; the last layer alone runs twice.
# R: a width and sizes that are multiples of 4 only, a map whose size is odd multiples of 2.
CONFIGS = {
    "K": {"architecture": "Ferodra", "vocab": 211, "width": 96, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 2},
          "layers": [
        layer(delta(6, 2, 24, 40, 4), moe(5, 1, 2, 48, 1.7, shared=40)),
        layer(attention(6, 2, 16, 24, 0.3, 0.45, softcap=4.0, rotation=rot(8, 3000.0, factor=8.0, original=64, fast=6.0, slow=0.5)), None),
        layer(attention(4, 4, 24, 16, 0.25, 0.2, softcap=20.0, rotation=rot(24, 10000.0, factor=4.0, original=32, fast=16.0, slow=2.0)),
              moe(6, 3, 3, 32, 0.8)),
        layer(delta(3, 3, 16, 8, 2), dense(72))]},
    "L": {"architecture": "Ferodra", "vocab": 300, "width": 128, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 2, "times": 3},
          "layers": [
        layer(attention(8, 2, 64, 128, 0.12, 0.6, softcap=12.0, rotation=rot(32, 500000.0, factor=2.0, original=64, fast=8.0, slow=1.0)),
              moe(8, 2, 2, 64, 2.5, shared=96)),
        layer(delta(4, 2, 32, 64, 4), dense(96)),
        layer(attention(4, 4, 64, 128, 0.2, 0.35, rotation=rot(64, 10000.0)), moe(4, 1, 1, 64, 1.0, shared=32))]},
    "M": {"architecture": "Ferodra", "vocab": 97, "width": 64, "norm": {"eps": 1e-6}, "layers": [
        layer(attention(1, 1, 8, 12, 0.5, 0.1), moe(2, 0, 2, 32, 1.0, shared=16)),
        layer(delta(1, 1, 160, 16, 1), None),
        layer(attention(2, 1, 32, 40, 0.2, 0.7, softcap=50.0, rotation=rot(16, 100.0)), dense(40)),
        layer(delta(2, 1, 8, 20, 5), moe(3, 2, 5, 16, 0.5))]},
    "N": {"architecture": "Ferodra", "vocab": 331, "width": 256, "norm": {"eps": 1e-6}, "loop": {"start": 2, "stop": 3, "times": 2},
          "layers": [
        layer(attention(4, 1, 64, 128, 0.15, 0.5, softcap=25.0, rotation=rot(48, 1000000.0, factor=4.0, original=256, fast=32.0, slow=1.0)),
              dense(160)),
        layer(delta(2, 1, 128, 128, 4), moe(6, 2, 2, 64, 1.2, shared=128)),
        layer(attention(6, 3, 64, 128, 0.1, 0.25, softcap=15.0), None)]},
    "R": {"architecture": "Ferodra", "vocab": 150, "width": 100, "norm": {"eps": 1e-5}, "loop": {"start": 0, "stop": 1, "times": 1},
          "layers": [
        layer(attention(5, 1, 22, 12, 0.3, 0.3, softcap=8.0, rotation=rot(10, 1000.0, factor=3.0, original=16, fast=4.0, slow=1.0)),
              moe(3, 1, 2, 36, 1.5, shared=20)),
        layer(delta(5, 5, 20, 12, 3), dense(44)),
        layer(delta(4, 2, 12, 20, 3), moe(3, 2, 2, 20, 1.5))]},
}
BLOCK_SIZE = {"K": 16, "L": 8, "M": 32, "N": 16, "R": 16}
SEED = {"K": 51, "L": 52, "M": 53, "N": 54, "R": 55}


def write_case(tmp_path, name: str, store_dtype=torch.bfloat16, std: float = 0.1, config=None, router_step: float = 0.0) -> str:
    """A model folder of configuration ``name`` with random weights.  ``std`` is large enough that attention weights, gates and
    decays are far from uniform.  ``router_step`` > 0: the routers' corrections are set that far apart
    (``spread_corrections``)."""
    from iian_b200.config.registry import get_architecture
    from iian_b200.weights.random_init import write_model_folder
    arch = get_architecture("Ferodra")
    d = os.path.join(str(tmp_path), f"ferodra{name}_{str(store_dtype).split('.')[-1]}" + ("_steady" if router_step else ""))
    if not os.path.isdir(d):
        write_model_folder(d, arch, arch.load_config(config or CONFIGS[name]), seed=SEED.get(name, 1), store_dtype=store_dtype,
                           std=std, norm_jitter=0.4)
        if router_step:
            spread_corrections(d, store_dtype, router_step)
    return d


def spread_corrections(model_dir: str, store_dtype, step: float) -> None:
    """Random router weights put the choice scores of a few experts within a hair of each other for a good part of the tokens,
    and 16-bit rounding of the router's input then decides which expert a token takes: another expert is another output at full
    size.  So for the bfloat16 runs of whole models the corrections are set ``step`` apart, in a shuffled order that differs from
    layer to layer: no choice is close.  The weights stay the softmax the input moves freely; the 32-bit runs and the kernels'
    own tests keep free choices too."""
    from iian_b200.weights.safetensors_io import write_safetensors
    w = plain.read_safetensors(os.path.join(model_dir, "model.safetensors"))
    for i, name in enumerate(sorted(k for k in w if k.endswith(".correction"))):
        n = w[name].numel()
        order = torch.randperm(n, generator=torch.Generator().manual_seed(200 + i)).to(torch.float32)
        w[name] = (order - (n - 1) / 2) * step
    write_safetensors(os.path.join(model_dir, "model.safetensors"),
                      {k: (v.to(store_dtype) if v.is_floating_point() else v) for k, v in w.items()}, metadata={"format": "pt"})


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
    return torch.tanh(addend.alpha * addend.y.double()) * addend.weight.double() + addend.bias.double()
