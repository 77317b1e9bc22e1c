"""Fezozen without a GPU: the configuration, the plan against the checkpoint layout, what the runs of
the layers ask of the cache, and the plain implementation's mechanisms against hand-worked numbers."""
import copy
import math

import numpy as np
import pytest

import plain_fezozen as plain
from tiny_configs import FEZOZEN_A, FEZOZEN_B, FEZOZEN_C


def _model(raw, dtype="float32"):
    from gemmars_b200.config.registry import resolve_architecture
    from gemmars_b200.engine.model import DecoderModel
    arch = resolve_architecture(raw)
    cfg = arch.config_class.from_dict(raw)
    return arch, cfg, DecoderModel(arch.build_plan(cfg, None), dtype, "cpu")


def test_configuration_reports_every_problem_at_once():
    from gemmars_b200.config.base import ConfigError
    from gemmars_b200.models.fezozen import FezozenConfig
    cfg = FezozenConfig.from_dict(FEZOZEN_A)
    assert cfg.vocab == 211 and cfg.embedding_scale == 3.0 and cfg.norm_eps == 1e-5 and len(cfg.layers) == 6
    assert FezozenConfig.from_dict(cfg.to_dict()) == cfg
    bad = copy.deepcopy(FEZOZEN_A)
    bad["layers"][0]["mixer"]["kv_heads"] = 4                      # 6 heads
    bad["layers"][0]["mlp"]["router"]["top"] = 6                   # of 5 experts
    bad["layers"][1]["mixer"]["rot"]["dims"] = 14                  # more than rot_dim
    del bad["layers"][1]["mixer"]["kv_rank"]
    bad["layers"][2]["mixer"]["rot"]["scaling"]["slow"] = 0
    bad["layers"][2]["mlp"]["kind"] = "dense"
    bad["layers"][3]["weights_of"] = 2                             # another kind of layer
    bad["layers"][4]["mixer"]["mask"]["size"] = 0
    bad["layers"][5]["type"] = "conv"
    del bad["embedding"]
    with pytest.raises(ConfigError) as e:
        FezozenConfig.from_dict(bad)
    for piece in ("6 heads", "top: 6 of 5", "layers[1].mixer.rot.dims", "mixer.kv_rank", "scaling.slow", "unknown feed-forward 'dense'",
                  "layers[3].weights_of", "mask.size", "unknown mixer 'conv'", "embedding.scale"):
        assert piece in str(e.value), piece
    circle = copy.deepcopy(FEZOZEN_A)
    circle["layers"][1]["weights_of"] = 3
    with pytest.raises(ConfigError, match="circle"):
        FezozenConfig.from_dict(circle)


def test_optional_entries_may_be_null_or_absent():
    from gemmars_b200.models.fezozen import FezozenConfig
    raw = copy.deepcopy(FEZOZEN_C)
    for layer in raw["layers"]:
        layer["weights_of"] = None
        layer["mixer"].setdefault("softcap", None)
        layer["mixer"].setdefault("mask", None)
        layer["mixer"]["rot"]["scaling"] = None
    cfg = FezozenConfig.from_dict(raw)
    assert all("weights_of" not in layer for layer in cfg.layers)
    assert _model(raw)[2].expected_tensors() == _model(FEZOZEN_C)[2].expected_tensors()
    del raw["layers"][2]["mlp"]
    assert FezozenConfig.from_dict(raw).layers[2].get("mlp") is None


@pytest.mark.parametrize("raw", [FEZOZEN_A, FEZOZEN_B, FEZOZEN_C], ids="ABC")
def test_plan_wants_exactly_the_checkpoint(raw):
    arch, cfg, model = _model(raw)
    layout = {name: tuple(shape) for name, (shape, _) in arch.checkpoint_layout(cfg).items()}
    assert model.expected_tensors() == layout
    for i, layer in enumerate(raw["layers"]):
        mine = [n for n in layout if n.startswith(f"l{i}.")]
        if "weights_of" in layer:
            assert not mine
            continue
        assert (f"l{i}.mix.q.b" in layout) == (layer["type"] == "attention")
        assert (f"l{i}.mix.g" in layout) == (layer["type"] == "latent_attention")
        if layer["mlp"] is None:
            assert f"l{i}.norm2" not in layout and {f"l{i}.norm2", f"l{i}.norm2b"} <= set(model.plan.ignored_tensors)


def test_shared_layers_are_runs_of_one_block_with_caches_of_their_own():
    from gemmars_b200.cache.pool import KVNeed
    _, _, model = _model(FEZOZEN_A)
    assert [e.layer for e in model.plan.schedule] == [0, 1, 2, 1, 0, 3] and len(model.blocks) == 4
    assert all(e.cache_of is None for e in model.plan.schedule)
    needs = dict(model.cache_needs())
    assert needs[0] == needs[4] == [KVNeed(2, 20, 20, 12)]             # a ring of the window's pages
    assert needs[1] == needs[3] == [KVNeed(1, 44 + 12, 33, 0)]         # one row of latent and rotated part, no values
    assert needs[2] == [KVNeed(4, 24, None, 28)] and needs[5] == [KVNeed(1, 20, None, 24)]
    # a layer may name the one that follows it, and one that itself names another
    raw = copy.deepcopy(FEZOZEN_A)
    raw["layers"][1]["weights_of"] = 3
    del raw["layers"][3]["weights_of"]
    assert [e.layer for e in _model(raw)[2].plan.schedule] == [0, 2, 1, 2, 0, 3]
    raw["layers"].append(dict(raw["layers"][1], weights_of=1))
    assert [e.layer for e in _model(raw)[2].plan.schedule] == [0, 2, 1, 2, 0, 3, 2]


def test_a_sublayer_stores_rows_that_are_its_own():
    """A sandwich block's parts write their output rows; the same parts in other blocks add to the stream."""
    from gemmars_b200.parts.base import build_part
    from gemmars_b200.parts.plan import PartSpec
    _, _, model = _model(FEZOZEN_A)
    for block in model.blocks:
        assert block.mixer.stores and (block.ffn is None or block.ffn.stores)
        assert block.chains_norms and block.first_norm() is block.mixer_norm
    spec = PartSpec("moe", {"hidden_size": 8, "experts": 2, "top": 1, "ff": 8})
    assert not build_part("ffn", spec, "float32").stores
    with pytest.raises(ValueError, match="without a gate"):
        build_part("ffn", PartSpec("moe", {**spec.params, "gated": False, "weigh": "input"}), "float32")


def test_the_rotations_frequencies():
    from gemmars_b200.parts.base import build_part
    for rot in (FEZOZEN_A["layers"][2]["mixer"]["rot"], FEZOZEN_A["layers"][5]["mixer"]["rot"], FEZOZEN_B["layers"][1]["mixer"]["rot"],
                {"base": 500.0, "dims": 8}, {"base": 1e6, "dims": 64, "scaling": {"factor": 3.0, "original": 10, "fast": 64.0, "slow": 32.0}}):
        from gemmars_b200.parts.plan import PartSpec
        part = build_part("position", PartSpec("rotary", {"head_dim": rot["dims"], "rotary_dim": rot["dims"], "theta": rot["base"],
                                                          "layout": "interleaved", "scaling": rot.get("scaling")}), "float32")
        f, stretch = plain.frequencies(rot["base"], rot["dims"], rot.get("scaling"))
        assert np.allclose(part.inv_freq("cpu").double().numpy(), f, rtol=1e-6) and part.magnitude == pytest.approx(stretch)


# ------------------------------------------------------------------ the mechanisms, by hand

def test_rotation_turns_neighbouring_dims():
    x = np.zeros((2, 1, 6))
    x[:, 0] = [1.0, 2.0, 3.0, 4.0, 5.0, 6.0]
    y = plain.rotate_pairs(x, [0, 1], {"base": math.pi ** -4.0, "dims": 4})      # f_0 = 1, f_1 = base^(-1/2) = pi^2
    assert np.allclose(y[0, 0], x[0, 0])
    c, s = math.cos(1.0), math.sin(1.0)
    c2, s2 = math.cos(math.pi ** 2), math.sin(math.pi ** 2)
    assert np.allclose(y[1, 0], [1 * c - 2 * s, 2 * c + 1 * s, 3 * c2 - 4 * s2, 4 * c2 + 3 * s2, 5.0, 6.0])


def test_scaled_frequencies_by_hand():
    # base e^2, 8 dims: the index of t turns is 2 ln(original / (2 pi t)); original = 2 pi e: 2 - 2 ln t
    base, original = math.exp(2.0), 2.0 * math.pi * math.e
    f, stretch = plain.frequencies(base, 8, {"factor": 5.0, "original": original, "fast": 2.0, "slow": 0.7})
    plain_f = np.exp(-0.5 * np.arange(4))
    # fast: 2 - 2 ln 2 = 0.61, floor 0; slow: 2 - 2 ln 0.7 = 2.71, ceil 3; the ramp is 0, 1/3, 2/3, 1
    mix = np.array([0.0, 1 / 3, 2 / 3, 1.0])
    assert np.allclose(f, plain_f * (1 - mix) + plain_f / 5.0 * mix) and stretch == pytest.approx(0.1 * math.log(5.0) + 1.0)
    # both ends on one index (floor 1.5, ceil 0.5): the ramp is a step there
    f, _ = plain.frequencies(base, 8, {"factor": 5.0, "original": original, "fast": math.e ** 0.25, "slow": math.e ** 0.75})
    assert np.allclose(f[:2], plain_f[:2]) and np.allclose(f[2:], plain_f[2:] / 5.0)


def test_the_window_keeps_its_size_with_the_token_itself():
    seen = plain.visible(6, 3)
    assert [list(np.nonzero(row)[0]) for row in seen] == [[0], [0, 1], [0, 1, 2], [1, 2, 3], [2, 3, 4], [3, 4, 5]]
    assert plain.visible(4, 1).tolist() == np.eye(4, dtype=bool).tolist()
    assert plain.visible(4, None).tolist() == np.tril(np.ones((4, 4), bool)).tolist()


def test_scores_are_scaled_then_capped():
    q, k = np.full((2, 1, 1), 2.0), np.array([[[10.0]], [[-10.0]]])
    v = np.array([[[1.0]], [[0.0]]])
    out = plain.masked_attention(q, k, v, 0.5, 4.0, None)
    a, b = 4 * math.tanh(10 / 4.0), 4 * math.tanh(-10 / 4.0)
    assert out[0, 0, 0] == 1.0 and out[1, 0, 0] == pytest.approx(1 / (1 + math.exp(b - a)))


def test_unit_queries_and_keys_come_after_the_rotation_and_over_every_dim():
    """With a stretched rotation of half the dims the order matters: the norm sees the stretched pair."""
    rng = np.random.default_rng(3)
    m = {"heads": 1, "kv_heads": 1, "dim": 4, "vdim": 2, "scale": 1.0, "mask": {"size": 8},
         "rot": {"base": 100.0, "dims": 2, "scaling": {"factor": 1e6, "original": 64, "fast": 4.0, "slow": 1.0}}}
    P = {k: rng.standard_normal(s) for k, s in (("q", (4, 5)), ("k", (4, 5)), ("v", (2, 5)), ("o", (3, 2)))}
    h = rng.standard_normal((3, 5))
    x = plain.rotate_pairs((h @ P["k"].T)[:, None], np.arange(3), m["rot"])
    assert np.allclose(np.mean(plain.unit_rms(x, 0.0) ** 2, axis=-1), 1.0)
    before = plain.rotate_pairs(plain.unit_rms((h @ P["k"].T)[:, None], 0.0), np.arange(3), m["rot"])
    assert np.abs(plain.unit_rms(x, 0.0) - before).max() > 0.1
    q = plain.unit_rms(plain.rotate_pairs((h @ P["q"].T)[:, None], np.arange(3), m["rot"]), 1e-3)
    want = plain.masked_attention(q, plain.unit_rms(x, 1e-3), (h @ P["v"].T)[:, None], 1.0, None, 8)[:, 0] @ P["o"].T
    assert np.allclose(plain.unit_attention_mixer(h, P, m, 1e-3), want)


def test_one_gate_per_number():
    rng = np.random.default_rng(0)
    m = {"heads": 2, "dim": 3, "rot_dim": 2, "vdim": 2, "kv_rank": 4, "scale": 0.5, "mask": {"size": 4}, "rot": {"base": 10.0, "dims": 2}}
    P = {k: rng.standard_normal(s) for k, s in (("q", (10, 6)), ("dkv", (6, 6)), ("uk", (6, 4)), ("uv", (4, 4)), ("g", (4, 6)))}
    P.update({"o": np.eye(4), "dkv.norm": np.ones(4)})
    h = rng.standard_normal((1, 6))
    c = plain.unit_rms(h @ P["dkv"][:4].T, 1e-6)
    # one key: its value, number by number through its own gate
    assert np.allclose(plain.latent_attention_mixer(h, P, m, 1e-6), (c @ P["uv"].T) / (1 + np.exp(-h @ P["g"].T)))


def test_scores_choose_and_weigh_the_input():
    z = np.log(np.array([0.2, 0.5, 0.8, 0.6]) / (1 - np.array([0.2, 0.5, 0.8, 0.6])))        # scores 0.2, 0.5, 0.8, 0.6
    chosen, s = plain.choose(z, 2)
    assert chosen == [2, 3] and np.allclose(s, [0.8, 0.6])                                    # not renormalized
    assert plain.choose(np.zeros(3), 2)[0] == [0, 1]                                          # the lower index wins a tie
    rng = np.random.default_rng(1)
    P = {"router": np.zeros((2, 3))}
    for e in range(2):
        P.update({f"e{e}.gate": rng.standard_normal((4, 3)), f"e{e}.up": rng.standard_normal((4, 3)), f"e{e}.down": rng.standard_normal((3, 4))})
    h = rng.standard_normal((1, 3))
    got = plain.routed_ffn(h, P, {"router": {"experts": 2, "top": 2}})
    assert np.allclose(got, plain.expert(0.5 * h, P, 0) + plain.expert(0.5 * h, P, 1))
    assert np.abs(got - 0.5 * (plain.expert(h, P, 0) + plain.expert(h, P, 1))).max() > 1e-3   # not the same as on the output


def test_sublayers_pass_a_norm_on_both_sides():
    """A layer's step into the stream is its norm's: as long as the norm's weight says, whatever the sublayer's size."""
    from gemmars_b200.weights import random_weights
    w = {k: v.double().numpy() for k, v in random_weights(FEZOZEN_A, 3).items()}
    w["l1.mix.o"] = 1e3 * w["l1.mix.o"]                            # far above eps
    toks = list(np.random.default_rng(1).integers(0, 211, 12))
    ref, layers = plain.forward(FEZOZEN_A, w, toks, return_layers=True)
    assert len(layers) == 6
    step = layers[1] - layers[0]                                   # a layer without feed-forward: one norm's output
    assert np.allclose(np.mean((step / w["l1.norm1b"]) ** 2, axis=-1), 1.0, atol=1e-3)
    loud = {**w, "l1.mix.o": 7.0 * w["l1.mix.o"]}
    assert np.allclose(plain.forward(FEZOZEN_A, loud, toks), ref, atol=1e-3 * np.abs(ref).max())
    wide = {**w, "l1.norm1b": 2.0 * w["l1.norm1b"]}
    _, layers2 = plain.forward(FEZOZEN_A, wide, toks, return_layers=True)
    assert np.allclose(layers2[1] - layers2[0], 2.0 * step)
