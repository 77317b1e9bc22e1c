"""Mevuvik without a GPU: the configuration, the plan against the checkpoint layout, what the runs of
the layers ask of the cache, and the plain implementation's mechanisms against hand-worked numbers."""
import copy
import math

import numpy as np
import pytest

import plain_mevuvik as plain
from tiny_configs import MEVUVIK_A, MEVUVIK_B, MEVUVIK_C


def _model(raw, dtype="float32"):
    from gemmars_b200.config.registry import resolve_architecture
    from gemmars_b200.engine.model import DecoderModel
    arch = resolve_architecture(raw)
    cfg = arch.config_class.from_dict(raw)
    return arch, cfg, DecoderModel(arch.build_plan(cfg, None), dtype, "cpu")


def test_configuration_reports_every_problem_at_once():
    from gemmars_b200.config.base import ConfigError
    from gemmars_b200.models.mevuvik import MevuvikConfig
    cfg = MevuvikConfig.from_dict(MEVUVIK_A)
    assert cfg.vocab == 211 and cfg.residual_mult == 0.7 and cfg.logit_softcap == 9.0 and cfg.loop == (0, 2, 2)
    assert MevuvikConfig.from_dict(cfg.to_dict()) == cfg
    plain_cfg = MevuvikConfig.from_dict(MEVUVIK_C)
    assert plain_cfg.loop is None and plain_cfg.logit_softcap is None
    assert MevuvikConfig.from_dict(plain_cfg.to_dict()) == plain_cfg
    bad = copy.deepcopy(MEVUVIK_A)
    bad["layers"][0]["mixer"]["left"]["kv_heads"] = 2              # 3 heads
    bad["layers"][0]["mixer"]["right"]["gate_cap"] = 0
    bad["layers"][0]["mlp"]["router"]["top"] = 6                   # of 5 experts
    bad["layers"][1]["mixer"]["rot"]["dims"] = 14                  # more than rot_dim
    del bad["layers"][1]["mixer"]["q_rank"]
    bad["layers"][2]["mlp"]["kind"] = "gated"
    bad["layers"][3]["type"] = "conv"
    bad["loop"]["stop"] = 9
    del bad["residual_mult"]
    with pytest.raises(ConfigError) as e:
        MevuvikConfig.from_dict(bad)
    for piece in ("3 heads", "right.gate_cap", "top: 6 of 5", "rot.dims", "mixer.q_rank", "unknown feed-forward 'gated'",
                  "unknown mixer 'conv'", "loop: layers 0 to 9 of 4", "residual_mult"):
        assert piece in str(e.value), piece


@pytest.mark.parametrize("raw", [MEVUVIK_A, MEVUVIK_B, MEVUVIK_C], ids="ABC")
def test_plan_wants_exactly_the_checkpoint(raw):
    arch, cfg, model = _model(raw)
    layout = {name: tuple(shape) for name, (shape, _) in arch.checkpoint_layout(cfg).items()}
    assert model.expected_tensors() == layout
    for i, layer in enumerate(raw["layers"]):
        assert layout[f"l{i}.norm1"] == () and layout[f"l{i}.ls1"] == (raw["width"],)
        if layer["mlp"] is None:
            assert f"l{i}.norm2" not in layout and {f"l{i}.norm2", f"l{i}.ls2"} <= set(model.plan.ignored_tensors)
    assert ("loop.step" in layout) == ("loop" in raw)


def test_the_loop_is_runs_of_the_schedule():
    """A looped layer is one block with several entries, each with storage of its own; the vector of a
    pass stands before the pass's first entry alone."""
    for raw, order, starts in ((MEVUVIK_A, [0, 1, 0, 1, 2, 3], {0: 0, 2: 1}), (MEVUVIK_B, [0, 1, 2, 1, 2, 1, 2], {1: 0, 3: 1, 5: 2}),
                               (MEVUVIK_C, [0, 1, 2], {})):
        _, cfg, model = _model(raw)
        assert [e.layer for e in model.plan.schedule] == order and len(model.blocks) == len(raw["layers"])
        assert all(e.cache_of is None for e in model.plan.schedule)
        assert {i: p.row for i, p in enumerate(model.before) if p is not None} == starts
        assert [i for i, _ in plain.runs(raw)] == order
        assert {k: t for k, (_, t) in enumerate(plain.runs(raw)) if t is not None} == starts


def test_what_the_runs_keep_per_sequence():
    from gemmars_b200 import kernels
    from gemmars_b200.cache.pool import KVNeed, StateNeed
    _, _, model = _model(MEVUVIK_A)
    needs = dict(model.cache_needs())
    assert sorted(needs) == list(range(6))
    # the two-branch layer: keys of 20 with values of 24, a matrix a head, and a vector with a maximum a head
    assert needs[0] == needs[2] == [KVNeed(1, 20, None, 24), StateNeed((5, kernels.matrix_memory_floats(24, 12))),
                                    StateNeed((5, kernels.matrix_memory_aux_floats(24, 12)))]
    # the latent layer: one row of latent and rotated part per position, no values
    assert needs[1] == needs[3] == [KVNeed(1, 44 + 12, None, 0)] and needs[4] == [KVNeed(1, 32 + 8, None, 0)]
    assert kernels.matrix_memory_floats(24, 12) == 32 * 12 and kernels.matrix_memory_floats(130, 3) == 256 * 3
    assert kernels.matrix_memory_aux_floats(24, 12) == 32 + 4 and kernels.matrix_memory_aux_floats(64, 33) == 3 * 68


def test_one_number_norms_and_scales_are_spread_when_loaded():
    import torch
    from gemmars_b200.engine.model import build_model
    from gemmars_b200.weights import random_weights
    w = random_weights(MEVUVIK_A, 3)
    model = build_model(raw_config=MEVUVIK_A, tensors=dict(w), dtype="float32", device="cpu", compile_kernels=False)
    block = model.blocks[0]
    assert block.mixer_norm.weight.shape == (72,) and torch.all(block.mixer_norm.weight == w["l0.norm1"].float())
    assert torch.all(model.embedding.norm_weight == w["embed.norm"].float())
    # the residual's factor times the layer's own, handed to the last products of both branches and to the experts
    want = 0.7 * w["l0.ls1"].float()
    for _, branch in block.mixer.branches:
        assert torch.equal(branch.o.out_scale, want)
    assert torch.equal(block.ffn.out_scale, 0.7 * w["l0.ls2"].float())
    assert torch.equal(model.blocks[2].ffn.down.out_scale, 0.7 * w["l2.ls2"].float())
    assert torch.equal(model.before[2].vector, w["loop.step"][1].float())


# ------------------------------------------------------------------ the mechanisms, by hand

def test_one_number_norm():
    x = np.array([[3.0, 4.0]])
    assert np.allclose(plain.number_norm(x, 2.0, 0.0), x / math.sqrt(12.5) * 2.0)
    assert np.allclose(plain.number_norm(np.zeros((1, 2)), 2.0, 1e-6), 0.0)


def test_rotation_turns_pairs_half_the_part_apart():
    x = np.zeros((2, 1, 6))
    x[:, 0] = [1.0, 2.0, 3.0, 4.0, 5.0, 6.0]
    y = plain.rotate_half(x, [0, 1], (math.pi ** 2) ** -2.0, 4)      # f_0 = 1, f_1 = base^(-1/2) = pi^2
    assert np.allclose(y[0, 0], x[0, 0])
    c, s = math.cos(1.0), math.sin(1.0)
    c2, s2 = math.cos(math.pi ** 2), math.sin(math.pi ** 2)
    assert np.allclose(y[1, 0], [1 * c - 3 * s, 2 * c2 - 4 * s2, 3 * c + 1 * s, 4 * c2 + 2 * s2, 5.0, 6.0])


def test_matrix_memory_two_tokens_by_hand():
    # one head, dim 2, vdim 1
    q = np.array([[[1.0, 0.0]], [[1.0, 1.0]]])
    k = np.array([[[2.0, 1.0]], [[1.0, 0.0]]])
    v = np.array([[[3.0]], [[5.0]]])
    log_in, log_forget = np.array([[1.0], [-2.0]]), np.array([[-0.5], [-0.25]])
    o, (S, n, m) = plain.matrix_memory_scan(q, k, v, log_in, log_forget)
    # token 0: m = max(-0.5 + 0, 1) = 1, keep e^-1.5 of nothing, write e^0: S = (6, 3), n = (2, 1), n.q = 2
    assert o[0, 0, 0] == pytest.approx(6.0 / (2.0 + 1e-6))
    # token 1: m = max(-0.25 + 1, -2) = 0.75, keep e^0, write e^-2.75
    w = math.exp(-2.75)
    assert np.allclose(S[0, :, 0], [6 + 5 * w, 3.0]) and np.allclose(n[0], [2 + w, 1.0]) and m[0] == 0.75
    assert o[1, 0, 0] == pytest.approx((9 + 5 * w) / (3 + w + 1e-6))
    # the maximum starts at zero, not below: a faint first write stays faint, and the denominator is e^0
    o, (S, n, m) = plain.matrix_memory_scan(q[:1], k[:1], v[:1], np.array([[-4.0]]), np.array([[-3.0]]))
    assert m[0] == pytest.approx(-3.0)
    o, (S, n, m) = plain.matrix_memory_scan(q[:1], k[:1], v[:1], np.array([[-4.0]]), np.array([[-0.1]]))
    assert m[0] == pytest.approx(-0.1) and n[0, 0] == pytest.approx(2 * math.exp(-3.9))
    assert o[0, 0, 0] == pytest.approx(6 * math.exp(-3.9) / (math.exp(0.1) + 1e-6))
    # carried from the state it left
    first = plain.matrix_memory_scan(q[:1], k[:1], v[:1], log_in[:1], log_forget[:1])[1]
    again, _ = plain.matrix_memory_scan(q[1:], k[1:], v[1:], log_in[1:], log_forget[1:], state=first)
    assert again[0, 0, 0] == pytest.approx((9 + 5 * w) / (3 + w + 1e-6))


def test_the_gates_are_capped_before_the_sigmoid():
    assert np.allclose(plain.capped(np.array([0.0, 2.0, 1e9]), 2.0), [0.0, 2 * math.tanh(1.0), 2.0])
    assert np.allclose(plain.capped(np.array([3.0]), None), [3.0])
    assert np.allclose(plain.log_sigmoid(np.array([0.0, -800.0, 800.0])), [math.log(0.5), -800.0, 0.0])


def test_the_correction_moves_the_choice_and_not_the_weights():
    z = np.log(np.array([0.2, 0.5, 0.8, 0.6]) / (1 - np.array([0.2, 0.5, 0.8, 0.6])))        # scores 0.2, 0.5, 0.8, 0.6
    chosen, w = plain.route_sigmoid(z, np.zeros(4), 2, 3.0)
    assert chosen == [2, 3] and np.allclose(w, [3 * 0.8 / 1.4, 3 * 0.6 / 1.4])
    chosen, w = plain.route_sigmoid(z, np.array([1.0, 0.0, 0.0, 0.0]), 2, 3.0)
    assert chosen == [0, 2] and np.allclose(w, [3 * 0.2 / 1.0, 3 * 0.8 / 1.0])
    chosen, _ = plain.route_sigmoid(np.zeros(3), np.zeros(3), 2, 1.0)
    assert chosen == [0, 1]                                                                   # the lower index wins a tie


def test_feed_forward_squares_the_relu():
    P = {"up": np.array([[1.0, 0.0], [-1.0, 2.0]]), "down": np.array([[1.0, 10.0]])}
    assert np.allclose(plain.dense_ffn(np.array([[3.0, 1.0], [1.0, 3.0]]), P), [[9.0], [1.0 + 250.0]])


def test_one_gate_per_head():
    rng = np.random.default_rng(0)
    m = {"heads": 2, "kv_heads": 1, "dim": 3, "vdim": 2, "scale": 0.5}
    P = {"q": rng.standard_normal((6, 4)), "k": rng.standard_normal((3, 4)), "v": rng.standard_normal((2, 4)),
         "g": np.zeros((2, 4)), "o": np.eye(4)}
    h = rng.standard_normal((1, 4))
    assert np.allclose(plain.head_gated_attention_mixer(h, P, m), 0.5 * np.tile(h @ P["v"].T, 2))   # one key: its value, twice, half open
    P["g"] = np.vstack([1e4 * h, -1e4 * h])
    assert np.allclose(plain.head_gated_attention_mixer(h, P, m)[0], np.concatenate([(h @ P["v"].T)[0], [0.0, 0.0]]))


def test_every_pass_of_the_loop_has_its_own_state_and_vector():
    """The looped model against one with the passes written out as layers of their own, the pass's vector
    folded into nothing else: the same logits; without the vectors, or with the first alone, others."""
    from gemmars_b200.weights import random_weights
    w = {k: v.double().numpy() for k, v in random_weights(MEVUVIK_A, 3).items()}
    toks = list(np.random.default_rng(1).integers(0, 211, 24))
    ref, layers = plain.forward(MEVUVIK_A, w, toks, return_layers=True)
    assert len(layers) == 6
    flat = copy.deepcopy(MEVUVIK_A)
    del flat["loop"]
    order = [0, 1, 0, 1, 2, 3]
    flat["layers"] = [MEVUVIK_A["layers"][i] for i in order]
    copies = {k: v for k, v in w.items() if not k.startswith("l") or k == "loop.step"}
    for at, i in enumerate(order):
        copies.update({f"l{at}." + k[len(f"l{i}."):]: v for k, v in w.items() if k.startswith(f"l{i}.")})
    assert not np.allclose(plain.forward(flat, copies, toks), ref, atol=1e-3)
    stepped = dict(w, **{"loop.step": np.zeros((2, 72))})
    assert np.allclose(plain.forward(MEVUVIK_A, stepped, toks), plain.forward(flat, copies, toks), rtol=0, atol=1e-12)
    once = dict(w, **{"loop.step": np.vstack([w["loop.step"][0], w["loop.step"][0]])})
    assert not np.allclose(plain.forward(MEVUVIK_A, once, toks), ref, atol=1e-4)
