"""The Demavik design without a GPU: its configuration, its spec, its checkpoint names and shapes, what its
layers ask of the cache manager, and the plain implementation's own mechanisms against closed forms."""
import copy
import math

import numpy as np
import pytest
import torch

import demavik_configs as dc
import plain_demavik as plain


def _arch(cfg):
    from velox_b200.config.registry import architecture_of

    return architecture_of(cfg)


@pytest.mark.parametrize("name", list(dc.ALL))
def test_configuration_is_read_and_written_back(name):
    cfg = dc.ALL[name]
    arch = _arch(cfg)
    typed = arch.parse_config(cfg)
    again = typed.to_json_dict()
    for key in ("layers", "norm", "embedding", "vocab", "width", "residual_mult"):
        assert again[key] == cfg[key]
    assert arch.parse_config(again) == typed


def test_keys_that_may_be_left_out():
    arch = _arch(dc.SMALL)
    cfg = copy.deepcopy(dc.SMALL)
    cfg.pop("embedding")
    cfg.pop("residual_mult")
    for i in (2, 3, 5):
        cfg["layers"][i]["mixer"].pop("rot")
    typed = arch.parse_config(cfg)
    assert typed.bigram is None and typed.embedding_scale == 1.0 and typed.residual_mult == 1.0
    spec = arch.build_spec(typed)
    assert "bigram" not in spec.checkpoint_tensors() and spec.layers[2].position.kind == "none"
    assert "weight_scale" not in spec.layers[0].norms["mixer"].params


def test_what_the_configuration_refuses():
    from velox_b200.config.model_config import ConfigError

    arch = _arch(dc.SMALL)

    def broken(change):
        cfg = copy.deepcopy(dc.SMALL)
        change(cfg)
        with pytest.raises(ConfigError):
            arch.parse_config(cfg)

    broken(lambda c: c["layers"][0].update(type="mamba"))
    broken(lambda c: c["layers"][0]["mixer"].update(conv=0))
    broken(lambda c: c["layers"][0]["mixer"].pop("dt_rank"))
    broken(lambda c: c["layers"][1]["mixer"].update(tau=0.0))
    broken(lambda c: c["layers"][2]["mixer"].update(heads=3))                      # 3 heads on 2 key heads
    broken(lambda c: c["layers"][2]["mixer"].update(mask={"size": 8}))
    broken(lambda c: c["layers"][2]["mixer"]["rot"].update(dims=26))               # a head has 24
    broken(lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7))
    broken(lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("low"))
    broken(lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].update(high=0.5))   # below low
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=1))                    # no attention layer
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=3))                    # not an earlier one
    broken(lambda c: c["layers"][5]["mixer"].update(kv_from=3))                    # has no keys of its own
    broken(lambda c: c["layers"][5]["mixer"].update(dim=16, rot=None))             # other keys than layer 2's
    broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda c: c["layers"][0]["mlp"].update(shared={"ff": 8}))
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=7))                # of 6 experts
    broken(lambda c: c["embedding"]["bigram"].update(buckets=0))
    broken(lambda c: c["embedding"]["bigram"].update(mul_prev=1.5))
    broken(lambda c: c.pop("norm"))
    broken(lambda c: c.update(layers=[]))


def test_tensor_names_and_shapes():
    spec = dc.build_spec(dc.SMALL, rank=5)
    t = {name: tuple(src.shape) for name, src in spec.checkpoint_tensors().items()}
    assert t["embed"] == (120, 64) and t["bigram"] == (54, 64) and t["head"] == (120, 64) and t["final.norm"] == (64,)
    assert t["l0.mix.in"] == (192, 64) and t["l0.mix.conv"] == (96, 4) and t["l0.mix.conv.b"] == (96,)
    assert t["l0.mix.x"] == (30, 96) and t["l0.mix.dt"] == (96, 6) and t["l0.mix.dt.b"] == (96,)
    assert t["l0.mix.A_log"] == (96, 12) and t["l0.mix.D"] == (96,) and t["l0.mix.o"] == (64, 96)
    assert t["l1.mix.q"] == (48, 64) and t["l1.mix.v"] == (80, 64) and t["l1.mix.g"] == (80, 64) and t["l1.mix.norm"] == (40,)
    assert t["l1.mix.a1"] == (5, 64) and t["l1.mix.a2"] == (48, 5) and t["l1.mix.a2.b"] == (48,) and t["l1.mix.o"] == (64, 80)
    assert t["l2.mix.q"] == (96, 64) and t["l2.mix.q.b"] == (96,) and t["l2.mix.q.norm"] == (96,)
    assert t["l2.mix.k"] == (48, 64) and t["l2.mix.k.norm"] == (48,) and t["l2.mix.v"] == (40, 64) and t["l2.mix.v.b"] == (40,)
    assert t["l2.mix.o"] == (64, 80)
    assert t["l3.mix.q"] == (144, 64) and not any(n.startswith(("l3.mix.k", "l3.mix.v")) for n in t)
    assert t["l0.mlp.router"] == (6, 64) and t["l0.mlp.router.b"] == (6,) and t["l0.mlp.e5.gate"] == (40, 64)
    assert t["l0.mlp.e5.down"] == (64, 40) and "l0.mlp.e6.gate" not in t
    assert t["l0.norm1"] == (64,) and t["l0.norm2"] == (64,) and "l3.norm2" not in t
    assert set(spec.ignored_tensors) == {"l3.norm2", "l4.norm2"}


def test_the_size_that_only_the_checkpoint_gives(tmp_path):
    """The inner size of the decay's low-rank pair is read from a tensor's shape, layer by layer."""
    from velox_b200.weights.loader import Checkpoint, WeightError, check_checkpoint

    folder = str(tmp_path / "model")
    dc.write_folder(folder, dc.ODD, dc.make_weights(dc.ODD, seed=1, rank=5))
    arch = _arch(dc.ODD)
    typed = arch.parse_config(dc.ODD)
    checkpoint = Checkpoint(folder)
    sizes = arch.checkpoint_sizes(typed, lambda name: checkpoint.shape(name) if name in checkpoint else None)
    assert sizes == {"low_ranks": {2: 5, 4: 5}}
    check_checkpoint(checkpoint, arch.build_spec(typed, **sizes))
    with pytest.raises(WeightError):
        check_checkpoint(checkpoint, arch.build_spec(typed))


def test_random_weights_folder(tmp_path):
    from helpers import read_config, read_tensors, write_model

    folder = str(tmp_path / "random")
    write_model(folder, dc.SMALL, seed=3, dtype="bfloat16")
    tensors = read_tensors(folder)
    assert set(tensors) == set(dc.build_spec(dc.SMALL).checkpoint_tensors())
    assert read_config(folder)["layers"] == dc.SMALL["layers"]
    assert np.isfinite(plain.forward(dc.SMALL, dc.as_numpy(tensors), [1, 2, 3, 4, 5])).all()


def test_parts_and_their_parameters():
    spec = dc.build_spec(dc.SMALL, rank=8)
    assert [l.mixer.kind for l in spec.layers] == ["selective_scan", "gated_linear_attention", "attention", "attention",
                                                   "selective_scan", "attention"]
    assert all(l.block == "post_norm" for l in spec.layers)
    assert [e.cache_of for e in spec.schedule] == [None, None, None, 2, None, 2]
    assert spec.layers[0].norms["mixer"].params["weight_scale"] == 0.35
    assert "weight_scale" not in spec.final_norm.params
    own, reader = spec.layers[2].mixer.params, spec.layers[3].mixer.params
    assert (own["head_dim"], own["key_dim"], own["value_dim"]) == (32, 24, 20) and not own.get("keys_from_cache")
    assert reader["keys_from_cache"] and reader["num_heads"] == 6 and own["qk_norm"] == 1e-6
    # layers that rotate alike share one table
    assert spec.layers[2].position is spec.layers[3].position is spec.layers[5].position
    assert spec.layers[2].position.params["scaling"] == {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}
    experts = spec.layers[0].feed_forward
    assert experts.kind == "routed_experts" and experts.params["router"] == "softmax"
    names = [s.name for s in experts.weights["gate_up.weight"].sources][:4]
    assert names == ["l0.mlp.e0.gate", "l0.mlp.e0.up", "l0.mlp.e1.gate", "l0.mlp.e1.up"]
    assert spec.embedding.params["bigram"] == dc.SMALL["embedding"]["bigram"] and spec.embedding.params["scale"] == 2.0


def test_wavelength_scaling_of_the_rotation():
    """The part's table against the plain frequencies: below, inside and above the range, and a range of one point."""
    from velox_b200.parts.rope import RotaryHalf, stretch_long_waves

    for rot in (dc.SMALL_ROT, dc.rot(32, 200.0, (2.0, 2.0, 2.0, 40)), dc.rot(64, 500.0, (8.0, 1.0, 4.0, 256))):
        f = rot["base"] ** (-2.0 * np.arange(rot["dims"] // 2) / rot["dims"])
        want = plain.pair_frequencies(rot)
        waves = 2 * math.pi / f
        sc = rot["scaling"]
        assert (waves < sc["original"] / sc["high"]).any() and (waves > sc["original"] / sc["low"]).any()
        assert np.allclose(stretch_long_waves(torch.from_numpy(f), sc).numpy(), want, rtol=1e-12)
        part = RotaryHalf({"head_dim": rot["dims"], "theta": rot["base"], "max_position": 50, "scaling": sc}, {}, torch.float32,
                          torch.device("cpu"))
        assert np.allclose(part.cos.numpy()[37], np.cos(37 * want), atol=1e-6)
        assert np.allclose(part.sin.numpy()[37], np.sin(37 * want), atol=1e-6)


def test_long_wavelengths_against_closed_forms():
    sc = dict(factor=4.0, low=1.0, high=4.0, original=64)
    f = 2 * math.pi / np.array([10.0, 32.0, 100.0])      # below 16, inside 16 .. 64, above 64
    from velox_b200.parts.rope import stretch_long_waves

    got = stretch_long_waves(torch.from_numpy(f), sc).numpy()
    s = (64 / 32 - 1.0) / 3.0
    assert np.allclose(got, [f[0], (1 - s) * f[1] / 4 + s * f[1], f[2] / 4])


# ------------------------------------------------------------------ the plain mechanisms themselves
def test_plain_selective_scan_against_closed_forms():
    A = np.array([[-1.0, -2.0]])
    x, dt = np.array([[3.0], [5.0]]), np.array([[0.5], [0.25]])
    B, C = np.array([[1.0, 2.0], [0.0, 0.0]]), np.array([[1.0, 0.0], [0.0, 1.0]])
    y, S = plain.selective_scan(x, dt, A, B, C, np.array([10.0]))
    # the first token writes dt x B; the second writes nothing and decays what is there
    assert np.allclose(y[0], 1.5 + 30.0) and np.allclose(y[1], 3.0 * math.exp(-0.5) + 50.0)
    assert np.allclose(S, [[1.5 * math.exp(-0.25), 3.0 * math.exp(-0.5)]])
    # a step of nothing leaves the state as it is
    _, S0 = plain.selective_scan(x[:1], 0.0 * dt[:1], A, B[:1], C[:1], np.array([0.0]), S=np.array([[7.0, 8.0]]))
    assert np.allclose(S0, [[7.0, 8.0]])


def test_plain_gated_linear_attention_against_closed_forms():
    k, q, v = np.array([[0.6, 0.8]]), np.array([[1.0, 0.5]]), np.array([[2.0, -1.0, 0.5]])
    out, S = plain.gated_states(q, k, v, np.ones((1, 2)))
    assert np.allclose(S, np.outer(k[0], v[0])) and np.allclose(out[0], 1.0 * v[0])
    # the decay acts on the rows that belong to key channels, and the token's own write is not decayed
    S0 = np.array([[1.0, 2.0, 3.0], [0.5, -1.0, 4.0]])
    _, S1 = plain.gated_states(q, k, v, np.array([[0.5, 0.0]]), S=S0)
    assert np.allclose(S1, np.array([[0.5, 1.0, 1.5], [0.0, 0.0, 0.0]]) + np.outer(k[0], v[0]))
    m = {"heads": 1, "dim": 2, "tau": 4.0}
    W = {"a1": np.eye(2), "a2": np.eye(2), "a2.b": np.array([0.0, 1.0])}
    alpha = plain.gla_decay(np.array([[0.3, -2.0]]), W, "", m)
    sig = lambda z: 1.0 / (1.0 + math.exp(-z))
    assert np.allclose(alpha[0, 0], [sig(0.3) ** 0.25, sig(-1.0) ** 0.25])


def test_plain_pair_rows_norm_and_router():
    assert plain.bigram_rows([5, 17, 3], 11, 4, 3) == [11, (5 * 4 + 17 * 3) % 11, (17 * 4 + 3 * 3) % 11]
    assert plain.bigram_rows([2 ** 30, 2 ** 30], 10 ** 9 + 7, 10 ** 9, 10 ** 9)[1] == (2 ** 31 * 10 ** 9) % (10 ** 9 + 7)
    # one statistic over all heads, not one per head
    cfg_eps = 0.0
    x = np.array([[3.0, 4.0, 0.0, 0.0]])
    assert np.allclose(plain.rms_unit(x, cfg_eps), x / 2.5)
    W = {"router": np.eye(4), "router.b": np.array([0.0, 3.0, 0.0, -5.0])}
    (picks,) = plain.route(np.array([[1.0, 0.0, 2.0, 6.0]]), W, "", {"top": 2})
    # logits 1, 3, 2, 1: the bias counts in the choice and in the weights
    assert [e for e, _ in picks] == [1, 2] and np.allclose([w for _, w in picks], [1 / (1 + math.exp(-1)), 1 / (1 + math.exp(1))])


def test_plain_keys_of_another_layer():
    """A reader's logits do not change with the reader's place in the list of heads, only with its source's keys."""
    W = dc.as_numpy(dc.make_weights(dc.SMALL, seed=3, rank=8))
    base = plain.forward(dc.SMALL, W, [4, 9, 2, 7, 1])
    for name, matters in (("l2.mix.k", True), ("l3.mix.q", True)):
        other = dict(W)
        other[name] = W[name][::-1].copy()
        assert (np.abs(plain.forward(dc.SMALL, other, [4, 9, 2, 7, 1]) - base).max() > 1e-3) == matters


def test_model_registry_and_presets():
    from velox_b200.config.presets import MODEL_SIZES, model_size, with_layers
    from velox_b200.config.registry import supported_architectures

    assert "Demavik" in supported_architectures()
    for name in MODEL_SIZES:
        if name == "tiny-d" or name.startswith("demavik-"):
            for layers in (None, 2, 6, 11):
                cfg = model_size(name)
                cfg = cfg if layers is None else with_layers(cfg, layers)
                _arch(cfg).build_spec(_arch(cfg).parse_config(cfg)).validate()
    assert "tiny-d" in MODEL_SIZES and "demavik-1.5b" in MODEL_SIZES


def test_bytes_and_operations_of_a_layer():
    from velox_b200.cli import roofline
    from velox_b200.config.presets import model_size

    cfg = model_size("tiny-d")
    weights, cached = roofline.layer_bytes(cfg, 3, 50)
    assert weights > 0 and cached > 0
    more, _ = roofline.layer_bytes(cfg, 1, 50)
    assert more < weights        # fewer tokens name fewer experts
    assert roofline.layer_flops(cfg, 64, 0) > roofline.layer_flops(cfg, 32, 0) > 0
