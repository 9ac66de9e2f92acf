"""Rilonex without a GPU: configuration round trip, checkpoint naming, ranks read off the tensors, the constants the layer struct
carries, registry, and identities of the oracle's mechanisms (oracle/rilonex_oracle.py) that do not depend on the product path."""
import json
import math

import pytest
import torch

from oracle import rilonex_oracle as O
from pegainfer_b200.rilonex import RilonexConfig, iter_random_weights, weight_shapes, with_ranks

LEFT = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 10, "scale": 0.35, "rot": {"dims": 4, "base": 100.0}}
RIGHT = {"heads": 3, "kv_heads": 1, "dim": 5, "vdim": 7, "conv": 3}
CHAN = {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 3, "conv": 2}
LRU = {"width": 18, "blocks": 3, "conv": 4}
CFG = {"architecture": "Rilonex", "vocab": 50, "width": 24, "norm": {"eps": 1e-5}, "streams": 2, "layers": [
    {"type": "parallel", "mixer": {"left": LEFT, "right": RIGHT, "left_scale": 0.25, "right_scale": 1.75}, "mlp": {"kind": "dense", "ff": 20}},
    {"type": "rglru", "mixer": LRU, "mlp": None},
    {"type": "channel_delta", "mixer": CHAN, "mlp": {"kind": "dense", "ff": 9}}]}
RANKS = {"l2.mix.a1": (11, 24), "l2.mix.g1": (6, 24)}


def test_config_round_trip_and_tensor_names():
    c = RilonexConfig.from_dict(CFG)
    assert RilonexConfig.from_dict(json.loads(json.dumps(c.to_dict()))) == c
    assert json.loads(json.dumps(c.to_dict())) == CFG
    c = with_ranks(c, RANKS)
    assert (c.layers[2].delta.decay_rank, c.layers[2].delta.gate_rank) == (11, 6)
    s = weight_shapes(c)
    assert s["l0.mix.left.q"] == (24, 24) and s["l0.mix.left.k"] == (12, 24) and s["l0.mix.left.v"] == (20, 24) and s["l0.mix.left.o"] == (24, 40)
    assert s["l0.mix.left.talk"] == (4, 4) and s["l0.mix.left.pb"] == (4,) and s["l0.mix.left.g"] == (4, 24)
    assert s["l0.mix.right.q"] == (5, 24) and s["l0.mix.right.v.conv"] == (21, 3) and s["l0.mix.right.a"] == (3, 24) and s["l0.mix.right.dt_bias"] == (3,)
    assert s["l0.mix.right.g"] == (21, 24) and s["l0.mix.right.norm"] == (7,) and s["l0.mix.right.o"] == (24, 21)
    assert s["l1.mix.ra"] == (3, 6, 6) and s["l1.mix.ri.b"] == (3, 6) and s["l1.mix.y.b"] == (18,) and s["l1.mix.conv"] == (18, 4) and s["l1.mix.lam"] == (18,)
    assert s["l2.mix.a1"] == (11, 24) and s["l2.mix.a2"] == (32, 11) and s["l2.mix.g2"] == (12, 6) and s["l2.mix.dt_bias"] == (32,) and s["l2.mix.A_log"] == (4,)
    assert s["l2.hc2.mix"] == (2, 2) and s["l0.hc1.in"] == (2,) and s["l0.mlp.down"] == (24, 20)
    for absent in ("l1.norm2", "l1.hc2.in", "l1.mlp.gate", "l2.mix.a", "l2.mix.g", "l0.mix.right.a1"):
        assert absent not in s
    assert {n for n, _ in iter_random_weights(c)} == set(s)
    plain = dict(CFG)
    del plain["streams"]
    assert not any(".hc" in n for n in weight_shapes(with_ranks(RilonexConfig.from_dict(plain), RANKS)))


def test_ranks_must_come_with_the_checkpoint():
    c = RilonexConfig.from_dict(CFG)
    with pytest.raises(KeyError):
        with_ranks(c, {"l2.mix.a1": (11, 24)})
    with pytest.raises(KeyError):
        with_ranks(c, {})
    assert with_ranks(with_ranks(c, RANKS), {}) == with_ranks(c, RANKS)  # already known: nothing to read


def test_unknown_kinds_are_refused():
    for at, key, value in ((0, "type", "conv"), (0, "mlp", {"kind": "moe"})):
        bad = json.loads(json.dumps(CFG))
        bad["layers"][at][key] = value
        with pytest.raises(ValueError):
            RilonexConfig.from_dict(bad)


def test_layer_struct_carries_the_designs_constants():
    from pegainfer_b200.layered import ModelCfg
    from pegainfer_b200.rilonex import RilonexModel
    c = with_ranks(RilonexConfig.from_dict(CFG), RANKS)
    a, b, d = (RilonexModel.layer_struct(l) for l in c.layers)
    assert (a.mixer_kind, a.heads, a.kv_heads, a.dim, a.vdim, a.rot_dims, a.rot_base) == (6, 4, 2, 6, 10, 4, 100.0)
    assert (a.d_heads, a.d_kv_heads, a.d_dim, a.d_vdim, a.conv, a.decay_rank, a.gate_rank) == (3, 1, 5, 7, 3, 0, 0)
    assert (a.left_scale, a.right_scale, a.mlp_kind, a.ff, a.mlp_act) == (0.25, 1.75, 1, 20, 1) and math.isclose(a.scale, 0.35, rel_tol=1e-6)
    assert (b.mixer_kind, b.lru_width, b.lru_blocks, b.conv, b.lru_rate, b.mlp_kind, b.ff) == (5, 18, 3, 4, 8.0, 0, 0)
    assert (d.mixer_kind, d.d_heads, d.d_kv_heads, d.d_dim, d.d_vdim, d.conv, d.decay_rank, d.gate_rank) == (2, 4, 2, 8, 3, 2, 11, 6)
    assert all(l.weights_of == -1 for l in (a, b, d))
    mc = RilonexModel.model_struct(c, ModelCfg())
    assert (mc.block_kind, mc.streams) == (4, 2)


def test_registry_knows_the_design(tmp_path):
    from pegainfer_b200.registry import FLOAT32_CAPABLE, architecture_of
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert architecture_of(str(tmp_path)) == "Rilonex" and "Rilonex" in FLOAT32_CAPABLE
    from pegainfer_b200 import build
    for f in ("gqa_attention.cu", "gqa_mixed_attention.cu", "recurrent_mixers.cu", "gemm_batched_mma.cu", "residual32_ops.cu"):
        assert f in build.PARTS_OF["Rilonex"][0]
    assert "layered_host.cpp" in build.PARTS_OF["Rilonex"][1]


def weights(seed=0):
    return {n: t.float() for n, t in iter_random_weights(with_ranks(RilonexConfig.from_dict(CFG), RANKS), seed)}


def test_oracle_is_causal():
    w = weights()
    toks = torch.randint(0, 50, (30,), generator=torch.Generator().manual_seed(1)).tolist()
    trail = []
    full = O.forward(CFG, w, toks, trail)
    assert torch.allclose(O.forward(CFG, w, toks[:17]), full[:17], atol=1e-5)
    assert len(trail) == 3 and trail[0].shape == (30, 24)


def test_oracle_scores_mix_over_heads_and_weights_are_not_normalised():
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(5, 4, 6, generator=g), torch.randn(5, 2, 6, generator=g)
    plain = O.mixed_scores(q, k, 0.5, torch.eye(4))
    assert torch.allclose(plain[3, 4, 2], 0.5 * q[4, 3] @ k[2, 1])
    talk = torch.zeros(4, 4)
    talk[1, 0], talk[1, 3] = 2.0, -1.0
    mixed = O.mixed_scores(q, k, 0.5, talk)
    assert torch.allclose(mixed[1], 2.0 * plain[0] - plain[3]) and mixed[0].abs().max() == 0
    pos = torch.arange(5)
    p = O.logistic_weights(torch.zeros(1, 5, 5), torch.tensor([0.0]), pos, pos)
    assert torch.allclose(p.sum(-1), 0.5 * torch.arange(1.0, 6.0)[None])  # every visible key weighs one half
    assert O.logistic_weights(torch.zeros(1, 5, 5), torch.tensor([-30.0]), pos, pos).sum() < 1e-10


def test_oracle_rotation_turns_halves_and_keeps_relative_angles():
    rot = {"dims": 4, "base": 100.0}
    g = torch.Generator().manual_seed(4)
    q, k = torch.randn(1, 1, 6, generator=g), torch.randn(1, 1, 6, generator=g)
    a = (O.rotate_halves(q, torch.tensor([9]), rot) * O.rotate_halves(k, torch.tensor([5]), rot)).sum()
    b = (O.rotate_halves(q, torch.tensor([14]), rot) * O.rotate_halves(k, torch.tensor([10]), rot)).sum()
    assert torch.allclose(a, b, atol=1e-5)
    one = torch.tensor([[[0.0, 1.0, 0.0, 0.0, 7.0, 8.0]]])
    r = O.rotate_halves(one, torch.tensor([3]), rot)[0, 0]  # entry 1 pairs with entry 3 and turns at 100^(-1/2)
    assert torch.allclose(r, torch.tensor([0.0, math.cos(0.3), 0.0, math.sin(0.3), 7.0, 8.0]), atol=1e-6)


def test_oracle_recurrences_carry_their_state():
    w = weights()
    h = torch.randn(19, 24, generator=torch.Generator().manual_seed(5))
    for run in (lambda x, s: O.gated_linear_mixer(x, w, "l1.mix.", LRU, s), lambda x, s: O.delta_mixer(x, w, "l2.mix.", CHAN, 1e-5, True, s),
                lambda x, s: O.delta_mixer(x, w, "l0.mix.right.", RIGHT, 1e-5, False, s)):
        whole, _ = run(h, None)
        a, st = run(h[:8], None)
        b, st = run(h[8:9], st)
        c, _ = run(h[9:], st)
        assert torch.allclose(torch.cat([a, b, c]), whole, atol=1e-5)


def test_oracle_linear_unit_forgets_with_its_gate():
    u = torch.tensor([[2.0], [3.0]])
    lam = torch.tensor([0.5])
    sp = math.log1p(math.exp(0.5))
    out, S = O.linear_unit(u, torch.tensor([[0.1], [0.2]]), torch.tensor([[1.0], [0.25]]), lam)
    a0, a1 = math.exp(-8 * 0.1 * sp), math.exp(-8 * 0.2 * sp)
    s0 = math.sqrt(1 - a0 * a0) * 2.0           # the first token has no special case
    s1 = a1 * s0 + math.sqrt(1 - a1 * a1) * 0.25 * 3.0
    assert torch.allclose(out[:, 0], torch.tensor([s0, s1])) and torch.allclose(S, torch.tensor([s1]))


def test_oracle_delta_rule_replaces_a_keys_value_and_decays_channels():
    k = torch.tensor([[[1.0, 0.0]], [[1.0, 0.0]]])
    q = torch.tensor([[[1.0, 0.0]], [[1.0, 1.0]]])
    v = torch.tensor([[[3.0, -1.0]], [[5.0, 2.0]]])
    one = torch.ones(2, 1, 2)
    o, S = O.delta_rule(q, k, v, one, torch.ones(2, 1))
    assert torch.allclose(o[1, 0], v[1, 0])     # a full-strength write to the same key replaces its value, and the read sees it
    S0 = torch.ones(1, 2, 2)
    g = torch.tensor([[[0.5, 0.25]]])
    o, S = O.delta_rule(torch.tensor([[[1.0, 0.0]]]), k[:1], v[:1], g, torch.zeros(1, 1), S0)
    assert torch.allclose(S[0], torch.tensor([[0.5, 0.5], [0.25, 0.25]])) and torch.allclose(o[0, 0], torch.tensor([0.5, 0.5]))


def test_oracle_streams_mix_from_the_old_rows():
    x = torch.tensor([[[1.0]], [[10.0]]])       # two streams, one token, one entry
    mix = torch.tensor([[0.5, 2.0], [3.0, 0.0]])  # [from, to]
    y = O.write_streams(x, torch.tensor([[100.0]]), mix, torch.tensor([1.0, -1.0]))
    assert y.flatten().tolist() == [0.5 + 30.0 + 100.0, 2.0 + 0.0 - 100.0]
    assert O.read_streams(x, torch.tensor([2.0, 0.1])).item() == 3.0
