"""``Demavik`` as a model spec.

The embedding times a constant, plus a row of a second table picked by (previous token, token), starts the float32
stream x; a layer is

    x <- x + m * norm1(mixer(x));   x <- x + m * norm2(experts(x))        (a layer may have no experts)

with m a constant of the model and every norm an RMS norm with a weight per coordinate: the norms sit on the
sublayers' results, the sublayers read x as it is.  The mixer is one of three, listed layer by layer:

* ``mamba1``: a selective scan behind a short convolution;
* ``gla``: gated linear attention with a decay per head and key channel;
* ``attention``: causal softmax attention, queries and keys normed over the whole projection and rotated; with
  ``kv_from`` the layer reads the keys and values that another layer has cached.

The experts are ``W_down (silu(W_gate h) * (W_up h))``, the ``top`` with the largest router logits, weighted by the softmax
over those.  After the last layer: norm and a head of its own.

This module only maps configuration keys to part parameters and checkpoint names to part
weights.  It has no forward pass.
"""
from __future__ import annotations

from typing import Dict, Optional

from ..config.model_config import (DemavikConfig, GatedLinearConfig, LongWaveRotation, ModelConfig, NormedAttentionConfig,
                                   SelectiveScanConfig, SoftmaxExpertsConfig)
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry, TensorSource, WeightSpec

ARCHITECTURE = "Demavik"


def _matrix(*sources: TensorSource) -> WeightSpec:
    return WeightSpec(sources=tuple(sources), role="matrix")


def _vector(*sources: TensorSource) -> WeightSpec:
    return WeightSpec(sources=tuple(sources), role="vector")


def _ones(name: str, size: int) -> WeightSpec:
    return _vector(TensorSource(name, (size,), init="one_plus_normal"))


def _rms(name: str, size: int, eps: float, scale: float = 1.0) -> PartSpec:
    params: Dict = {"size": size, "eps": eps}
    if scale != 1.0:
        params["weight_scale"] = scale
    return PartSpec(kind="rms", params=params, weights={"weight": _ones(name, size)})


def _scan(prefix: str, m: SelectiveScanConfig, width: int) -> PartSpec:
    I, N, R = m.inner, m.state, m.dt_rank
    return PartSpec(
        kind="selective_scan",
        params={"hidden_size": width, "inner": I, "state_size": N, "rank": R, "conv_taps": m.conv},
        weights={
            "in.weight": _matrix(TensorSource(prefix + "in", (2 * I, width))),
            "conv.weight": _vector(TensorSource(prefix + "conv", (I, m.conv), init="uniform:-0.6:0.6")),
            "conv.bias": _vector(TensorSource(prefix + "conv.b", (I,))),
            "low.weight": _matrix(TensorSource(prefix + "x", (R + 2 * N, I))),
            "dt.weight": _matrix(TensorSource(prefix + "dt", (I, R))),
            "dt.bias": _vector(TensorSource(prefix + "dt.b", (I,), init="uniform:-5:-2")),
            "a_log": _vector(TensorSource(prefix + "A_log", (I, N), init="uniform:0:2.7")),
            "d": _vector(TensorSource(prefix + "D", (I,), init="one_plus_normal")),
            "out.weight": _matrix(TensorSource(prefix + "o", (width, I))),
        })


def default_rank(m: GatedLinearConfig) -> int:
    """The inner size of a ``gla`` layer's low-rank pair where no checkpoint gives it."""
    return 16


def _linear(prefix: str, m: GatedLinearConfig, width: int, eps: float, rank: int) -> PartSpec:
    keys, inner = m.heads * m.dim, m.heads * m.vdim
    return PartSpec(
        kind="gated_linear_attention",
        params={"hidden_size": width, "heads": m.heads, "dim": m.dim, "value_dim": m.vdim, "rank": rank, "tau": m.tau,
                "eps": eps},
        weights={
            "in.weight": _matrix(TensorSource(prefix + "q", (keys, width)), TensorSource(prefix + "k", (keys, width)),
                                 TensorSource(prefix + "v", (inner, width)), TensorSource(prefix + "g", (inner, width)),
                                 TensorSource(prefix + "a1", (rank, width))),
            "decay_up.weight": _matrix(TensorSource(prefix + "a2", (keys, rank), init="normal_wide")),
            "decay_bias": _vector(TensorSource(prefix + "a2.b", (keys,), init="normal_wide")),
            "norm.weight": _ones(prefix + "norm", m.vdim),
            "out.weight": _matrix(TensorSource(prefix + "o", (width, inner))),
        })


def _attention(prefix: str, m: NormedAttentionConfig, width: int, eps: float, head_dim: int) -> PartSpec:
    H, G = m.heads, m.kv_heads
    params = {"hidden_size": width, "num_heads": H, "num_kv_heads": G, "head_dim": head_dim, "key_dim": m.dim,
              "value_dim": m.vdim, "softmax_scale": m.scale, "qkv_bias": True, "qk_norm": eps}
    weights = {
        "q.weight": _matrix(TensorSource(prefix + "q", (H * m.dim, width))),
        "q.bias": _vector(TensorSource(prefix + "q.b", (H * m.dim,))),
        "q_norm": _ones(prefix + "q.norm", H * m.dim),
        "out.weight": _matrix(TensorSource(prefix + "o", (width, H * m.vdim))),
    }
    if m.kv_from is not None:
        params["keys_from_cache"] = True
    else:
        for name, size in (("k", m.dim), ("v", m.vdim)):
            weights[f"{name}.weight"] = _matrix(TensorSource(prefix + name, (G * size, width)))
            weights[f"{name}.bias"] = _vector(TensorSource(f"{prefix}{name}.b", (G * size,)))
        weights["k_norm"] = _ones(prefix + "k.norm", G * m.dim)
    return PartSpec(kind="attention", params=params, weights=weights)


def _position(rot: Optional[LongWaveRotation], head_dim: int, max_position: int) -> PartSpec:
    if rot is None:
        return PartSpec(kind="none", params={"head_dim": head_dim})
    params = {"head_dim": head_dim, "rotary_dim": rot.dims, "theta": rot.base, "max_position": max_position,
              "angles": "float64"}
    if rot.scaling is not None:
        params["scaling"] = dict(zip(("factor", "low", "high", "original"), rot.scaling))
    return PartSpec(kind="rotary_half", params=params)


def _experts(prefix: str, f: SoftmaxExpertsConfig, width: int) -> PartSpec:
    X, F = f.experts, f.ff
    return PartSpec(
        kind="routed_experts",
        params={"hidden_size": width, "experts": X, "top": f.top, "expert_ff": F, "router": "softmax"},
        weights={
            "router.weight": _matrix(TensorSource(prefix + "router", (X, width))),
            "router.correction": _vector(TensorSource(prefix + "router.b", (X,))),
            "gate_up.weight": _matrix(*(TensorSource(f"{prefix}e{e}.{name}", (F, width))
                                        for e in range(X) for name in ("gate", "up"))),
            "down.weight": _matrix(*(TensorSource(f"{prefix}e{e}.down", (width, F)) for e in range(X))),
        })


def build_demavik_spec(config: ModelConfig, low_ranks: Optional[Dict[int, int]] = None) -> ModelSpec:
    """``low_ranks``: per ``gla`` layer the inner size of the decay's pair of matrices.  No configuration key names it: a
    checkpoint's tensor shapes do (``checkpoint_sizes``, which the loader of a model folder calls); without a
    checkpoint it is ``default_rank``."""
    if not isinstance(config, DemavikConfig):
        raise TypeError(f"expected a DemavikConfig, got {type(config).__name__}")
    c = config
    E, V, m = c.hidden_size, c.vocab_size, c.residual_mult
    layers, schedule = [], []
    positions: Dict = {}  # layers that rotate alike share their tables
    for index, layer in enumerate(c.layers):
        p = f"l{index}."
        position = cache_of = None
        if layer.scan is not None:
            mixer = _scan(p + "mix.", layer.scan, E)
        elif layer.linear is not None:
            rank = (low_ranks or {}).get(index, default_rank(layer.linear))
            mixer = _linear(p + "mix.", layer.linear, E, c.norm_eps, rank)
        else:
            a = layer.attention
            # Heads padded with zeros to a size the attention kernels take.
            head_dim = -(-max(a.dim, a.vdim) // 16) * 16
            mixer = _attention(p + "mix.", a, E, c.norm_eps, head_dim)
            key = (a.rot, head_dim)
            if key not in positions:
                positions[key] = _position(a.rot, head_dim, c.max_position_embeddings)
            position, cache_of = positions[key], a.kv_from
        norms = {"mixer": _rms(p + "norm1", E, c.norm_eps, m)}
        feed_forward = None
        if layer.mlp is not None:
            feed_forward = _experts(p + "mlp.", layer.mlp, E)
            norms["feed_forward"] = _rms(p + "norm2", E, c.norm_eps, m)
        layers.append(LayerSpec(block="post_norm", mixer=mixer, feed_forward=feed_forward, norms=norms, position=position))
        schedule.append(ScheduleEntry(layer=index, cache_of=cache_of))
    embedding = {"vocab_size": V, "hidden_size": E, "scale": c.embedding_scale}
    tables = {"weight": _matrix(TensorSource("embed", (V, E)))}
    if c.bigram is not None:
        embedding["bigram"] = c.bigram.to_json_dict()
        tables["bigram"] = _matrix(TensorSource("bigram", (c.bigram.buckets + 1, E)))
    spec = ModelSpec(
        architecture=c.architecture,
        hidden_size=E,
        vocab_size=V,
        max_position=c.max_position_embeddings,
        embedding=PartSpec(kind="token_embedding", params=embedding, weights=tables),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=_rms("final.norm", E, c.norm_eps),
        lm_head=PartSpec(kind="linear_head", params={"hidden_size": E, "vocab_size": V},
                         weights={"weight": _matrix(TensorSource("head", (V, E)))}),
        eos_token_ids=tuple(c.eos_token_ids),
        # A layer without feed-forward has no use for its norm; a file may still carry it.
        ignored_tensors=tuple(f"l{i}.norm2" for i, layer in enumerate(c.layers) if layer.mlp is None),
    )
    spec.validate()
    return spec


def checkpoint_sizes(config: ModelConfig, shape_of) -> Dict[str, Dict[int, int]]:
    """Sizes that only the checkpoint gives, as keyword arguments for ``build_demavik_spec``: ``shape_of(name)`` returns a
    tensor's shape or None."""
    ranks: Dict[int, int] = {}
    for index, layer in enumerate(config.layers):
        if layer.linear is not None:
            shape = shape_of(f"l{index}.mix.a1")
            if shape is not None and len(shape) == 2:
                ranks[index] = int(shape[0])
    return {"low_ranks": ranks}


register_architecture(ARCHITECTURE, DemavikConfig.from_dict, build_demavik_spec, checkpoint_sizes)
