"""Small Demavik configurations and weights for the tests.

The configurations differ in every size and make sizes differ that a model may happen to make
equal or 1: channels of the selective scan below, equal to and above the width, 1 to 200 states a channel,
step-size ranks of 1 and more, convolutions of 1 to 9 taps; key sizes and value sizes of the recurrent
heads (one below, equal to and above the other, multiples of four and not, above 128 and 256), one head,
several exponents of the decay; attention heads whose key and value sizes differ and are no multiples of
sixteen, one to six query heads per key head, rotations of some, most and all dims, with wavelengths on both
sides of the scaling's range and inside it, without scaling, layers that read an earlier layer's keys (with
another number of query heads than that layer has), one of them right behind it and one with layers in
between, two readers of one layer; one expert per token, some and all of them; layers without feed-forward;
widths and inner widths that are no multiples of eight; pair tables with products far above 32 bits, and
none; every order of the three kinds of layer.  ``make_weights`` draws weights at a scale at which every
mechanism does something: decays between forgetting in a few tokens and hardly at all, taps that reorder
what a token reads, router biases that change the choice.
"""
from __future__ import annotations

import json
import os
from typing import Any, Dict, Optional

import torch


def mamba(inner, state, dt_rank, conv) -> Dict[str, Any]:
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def gla(heads, dim, vdim, tau) -> Dict[str, Any]:
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def rot(dims, base=100.0, scaling=None) -> Dict[str, Any]:
    out: Dict[str, Any] = {"base": base, "dims": dims}
    if scaling is not None:
        out["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return out


def attn(heads, kv_heads, dim, vdim, scale, rotation, kv_from=None) -> Dict[str, Any]:
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rotation}
    if kv_from is not None:
        out["kv_from"] = kv_from
    return out


def moe(experts, top, ff) -> Dict[str, Any]:
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(kind, mixer, mlp) -> Dict[str, Any]:
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(width, vocab, layers, eps=1e-5, mult=0.4, scale=1.0, bigram: Optional[tuple] = (97, 31, 7)) -> Dict[str, Any]:
    embedding: Dict[str, Any] = {"scale": scale}
    if bigram is not None:
        embedding["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return {"architecture": "Demavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": embedding, "layers": layers}


# All three kinds of layer, a reader right behind its source and one further on with other query heads.
SMALL_ROT = rot(16, 60.0, (4.0, 1.0, 4.0, 64))
SMALL = config(64, 120, [
    layer("mamba1", mamba(96, 12, 6, 4), moe(6, 2, 40)),
    layer("gla", gla(2, 24, 40, 8.0), moe(5, 3, 24)),
    layer("attention", attn(4, 2, 24, 20, 0.3, SMALL_ROT), moe(4, 1, 32)),
    layer("attention", attn(6, 2, 24, 20, 0.25, SMALL_ROT, kv_from=2), None),
    layer("mamba1", mamba(64, 16, 8, 3), None),
    layer("attention", attn(2, 2, 24, 20, 0.35, SMALL_ROT, kv_from=2), moe(3, 3, 16)),
], eps=1e-6, mult=0.35, scale=2.0, bigram=(53, 1000003, 998244353))

# Widths that are no multiples of eight, sizes of one, no scaling of the rotation, no pair table.
ODD = config(100, 331, [
    layer("attention", attn(3, 1, 14, 30, 0.4, rot(10, 30.0)), moe(5, 2, 17)),
    layer("mamba1", mamba(54, 5, 3, 2), None),
    layer("gla", gla(3, 10, 7, 1.0), moe(7, 2, 20)),
    layer("attention", attn(6, 1, 14, 30, 0.3, rot(10, 30.0), kv_from=0), moe(2, 2, 9)),
    layer("gla", gla(1, 6, 15, 3.5), None),
    layer("mamba1", mamba(130, 1, 1, 1), moe(9, 4, 12)),
], eps=1e-5, mult=0.3, scale=1.3, bigram=None)

# Sizes near a real model's.
WIDE = config(256, 500, [
    layer("gla", gla(4, 64, 128, 16.0), moe(16, 4, 64)),
    layer("mamba1", mamba(512, 16, 16, 4), moe(8, 2, 96)),
    layer("attention", attn(8, 2, 64, 64, 0.125, rot(64, 500.0, (8.0, 1.0, 4.0, 256))), moe(12, 3, 64)),
    layer("attention", attn(4, 2, 64, 64, 0.125, rot(64, 500.0, (8.0, 1.0, 4.0, 256)), kv_from=2), moe(4, 2, 128)),
], eps=2e-5, mult=0.25, scale=4.0, bigram=(400, 7, 11))

# Large key sizes and many states, long convolutions, many query heads on one key head.
TALL = config(80, 200, [
    layer("mamba1", mamba(40, 40, 5, 9), moe(4, 2, 24)),
    layer("gla", gla(2, 136, 12, 12.0), None),
    layer("mamba1", mamba(24, 130, 2, 5), None),
    layer("attention", attn(6, 1, 32, 8, 0.2, rot(32, 200.0, (2.0, 2.0, 2.0, 40))), moe(3, 1, 16)),
    layer("gla", gla(1, 264, 36, 20.0), moe(4, 4, 8)),
    layer("mamba1", mamba(20, 200, 4, 4), None),
], eps=1e-6, mult=0.5, scale=0.7, bigram=(7, -5, 3))

ALL = {"small": SMALL, "odd": ODD, "wide": WIDE, "tall": TALL}

# The inner size of a gla layer's low-rank pair is a tensor shape, not a configuration key.
RANKS = {"small": 8, "odd": 5, "wide": 16, "tall": 20}


def build_spec(cfg: Dict[str, Any], rank: Optional[int] = None):
    from velox_b200.config.registry import architecture_of

    arch = architecture_of(cfg)
    ranks = None if rank is None else {i: rank for i, l in enumerate(cfg["layers"]) if l["type"] == "gla"}
    return arch.build_spec(arch.parse_config(cfg), low_ranks=ranks)


def make_weights(cfg: Dict[str, Any], seed: int, sharp: float = 1.0, rank: Optional[int] = None) -> Dict[str, torch.Tensor]:
    """Tensors under the checkpoint's names, bfloat16.  ``sharp`` scales the attention layers' query norms: at 2 or
    more the softmax puts most of its weight on a few keys."""
    spec = build_spec(cfg, rank)
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, source in sorted(spec.checkpoint_tensors().items()):
        shape = tuple(source.shape)
        rand = torch.randn(shape, generator=gen)
        last = name.split(".", 2)[-1] if name[1:2].isdigit() else name
        if name == "embed":
            t = rand / cfg["embedding"]["scale"]
        elif name == "bigram":
            t = 0.6 * rand
        elif last.endswith("norm") or last in ("norm1", "norm2"):
            t = 1.0 + 0.3 * rand
            if last == "q.norm":
                t = t * sharp
        elif last == "conv":
            t = 0.6 * rand
            t[:, -1] += 1.0
        elif last == "A_log":
            t = -0.5 + 0.8 * rand
        elif last == "dt.b":
            t = -2.0 + 1.2 * rand
        elif last == "a2.b":
            t = 2.0 + 2.0 * rand
        elif last == "D":
            t = 1.0 + 0.4 * rand
        elif last == "router.b":
            t = 0.7 * rand
        elif last.endswith(".b"):
            t = 0.5 * rand
        elif last == "router":
            t = 2.0 * rand / shape[-1] ** 0.5
        else:
            t = rand / shape[-1] ** 0.5
        out[name] = t.to(torch.bfloat16)
    return out


def write_folder(folder: str, cfg: Dict[str, Any], tensors: Dict[str, torch.Tensor]) -> None:
    from safetensors.torch import save_file

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as handle:
        json.dump(cfg, handle)
    save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(folder, "model.safetensors"))


def as_numpy(tensors: Dict[str, torch.Tensor]):
    return {k: v.double().numpy() for k, v in tensors.items()}
