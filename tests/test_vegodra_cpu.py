"""Vegodra without a GPU: configuration round trip, checkpoint naming, the rank read off the tensors, the constants the layer struct
carries, registry, and identities of the oracle's mechanisms (oracle/vegodra_oracle.py) that do not depend on the product path."""
import json
import math

import pytest
import torch

from oracle import vegodra_oracle as O
from pegainfer_b200.vegodra import VegodraConfig, iter_random_weights, weight_shapes, with_ranks

ATT = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 10, "mask": {"size": 7}, "scale": 0.35, "rot": {"dims": 4, "base": 100.0}}
LAT = {"heads": 3, "dim": 6, "rot_dim": 4, "vdim": 5, "q_rank": 9, "kv_rank": 11, "scale": 0.4, "rot": {"dims": 4, "base": 50.0}}
GLA = {"heads": 2, "dim": 5, "vdim": 7, "tau": 3.0}
CFG = {"architecture": "Vegodra", "vocab": 50, "width": 24, "norm": {"eps": 1e-5}, "layers": [
    {"type": "attention", "mixer": ATT, "mlp": {"kind": "dense", "ff": 20}},
    {"type": "latent_attention", "mixer": LAT, "mlp": None},
    {"type": "gla", "mixer": GLA, "mlp": {"kind": "dense", "ff": 9}},
    {"type": "attention", "mixer": dict(ATT, kv_from=0, mask={"size": 12}, scale=0.2), "mlp": {"kind": "dense", "ff": 13}}]}
RANKS = {"l2.mix.a1": (6, 24)}


def test_config_round_trip_and_tensor_names():
    c = VegodraConfig.from_dict(CFG)
    assert VegodraConfig.from_dict(json.loads(json.dumps(c.to_dict()))) == c
    assert json.loads(json.dumps(c.to_dict())) == CFG
    c = with_ranks(c, RANKS)
    assert c.layers[2].mixer.decay_rank == 6
    s = weight_shapes(c)
    assert s["embed.norm"] == s["embed.norm.b"] == s["l3.norm1.b"] == s["final.norm.b"] == (24,)
    assert s["l0.mix.q"] == (24, 24) and s["l0.mix.k"] == (12, 24) and s["l0.mix.v"] == (20, 24) and s["l0.mix.o"] == (24, 40)
    assert s["l0.mix.sink"] == (4,) and s["l0.mix.g"] == (4, 24) and s["l3.mix.g"] == (4, 24) and s["l3.mix.sink"] == (4,)
    assert s["l1.mix.dq"] == (9, 24) and s["l1.mix.dq.norm"] == (9,) and s["l1.mix.uq"] == (30, 9) and s["l1.mix.dkv"] == (15, 24)
    assert s["l1.mix.dkv.norm"] == (11,) and s["l1.mix.uk"] == (18, 11) and s["l1.mix.uv"] == (15, 11) and s["l1.mix.g"] == (15, 24) and s["l1.mix.o"] == (24, 15)
    assert s["l2.mix.a1"] == (6, 24) and s["l2.mix.a2"] == (10, 6) and s["l2.mix.a2.b"] == (10,) and s["l2.mix.norm"] == (7,) and s["l2.mix.g"] == (14, 24)
    assert s["l2.mlp.gate"] == (9, 24) and s["l2.mlp.down"] == (24, 9)
    for absent in ("l3.mix.k", "l3.mix.v", "l1.mlp.gate", "l1.mix.sink", "l0.norm2", "l1.mix.q"):
        assert absent not in s
    assert {n for n, _ in iter_random_weights(c)} == set(s)


def test_rank_must_come_with_the_checkpoint():
    c = VegodraConfig.from_dict(CFG)
    with pytest.raises(KeyError):
        with_ranks(c, {})
    assert with_ranks(with_ranks(c, RANKS), {}) == with_ranks(c, RANKS)  # already known: nothing to read


def test_unknown_kinds_are_refused():
    for at, key, value in ((0, "type", "conv"), (0, "mlp", {"kind": "moe"})):
        bad = json.loads(json.dumps(CFG))
        bad["layers"][at][key] = value
        with pytest.raises(ValueError):
            VegodraConfig.from_dict(bad)


def test_layer_struct_carries_the_designs_constants():
    from pegainfer_b200.layered import ModelCfg
    from pegainfer_b200.vegodra import VegodraModel
    c = with_ranks(VegodraConfig.from_dict(CFG), RANKS)
    a, l, g, b = (VegodraModel.layer_struct(x) for x in c.layers)
    assert (a.mixer_kind, a.heads, a.kv_heads, a.dim, a.vdim, a.chunk, a.rot_dims, a.rot_base, a.rot_interleaved) == (1, 4, 2, 6, 10, 7, 4, 100.0, 0)
    assert (a.sink_kind, a.out_gate, a.qk_norm, a.kv_from, a.mlp_kind, a.ff, a.mlp_act) == (0, 2, 3, -1, 1, 20, 2) and math.isclose(a.scale, 0.35, rel_tol=1e-6)
    assert (b.kv_from, b.chunk, b.ff) == (0, 12, 13) and math.isclose(b.scale, 0.2, rel_tol=1e-6)
    assert (l.mixer_kind, l.q_rank, l.kv_rank, l.rot_dim, l.rot_dims, l.rot_interleaved, l.sink_kind, l.out_gate, l.mlp_kind, l.kv_from) == (0, 9, 11, 4, 4, 1, 1, 1, 0, -1)
    assert (g.mixer_kind, g.heads, g.dim, g.vdim, g.tau, g.decay_rank, g.ff, g.kv_from) == (7, 2, 5, 7, 3.0, 6, 9, -1)
    assert all(x.weights_of == -1 and x.window == 0 and x.has_scaling == 0 for x in (a, l, g, b))
    assert VegodraModel.model_struct(c, ModelCfg()).block_kind == 5


def test_registry_knows_the_design(tmp_path):
    from pegainfer_b200.registry import FLOAT32_CAPABLE, architecture_of
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert architecture_of(str(tmp_path)) == "Vegodra" and "Vegodra" in FLOAT32_CAPABLE
    from pegainfer_b200 import build
    for f in ("gqa_attention.cu", "latent_attention.cu", "latent_attention_mma.cu", "recurrent_mixers.cu", "gemm_batched_mma.cu", "residual32_ops.cu"):
        assert f in build.PARTS_OF["Vegodra"][0]
    assert "layered_host.cpp" in build.PARTS_OF["Vegodra"][1]


def weights(seed=0):
    return {n: t.float() for n, t in iter_random_weights(with_ranks(VegodraConfig.from_dict(CFG), RANKS), seed)}


def test_oracle_is_causal_and_sums_both_sublayers_from_one_norm():
    w = weights()
    toks = torch.randint(0, 50, (30,), generator=torch.Generator().manual_seed(1)).tolist()
    trail = []
    full = O.forward(CFG, w, toks, trail)
    assert torch.allclose(O.forward(CFG, w, toks[:17]), full[:17], atol=1e-5)
    assert len(trail) == 4 and trail[0].shape == (30, 24)
    x0 = O.layer_norm(w["embed"][toks], w["embed.norm"], w["embed.norm.b"], 1e-5)
    h = O.layer_norm(x0, w["l0.norm1"], w["l0.norm1.b"], 1e-5)
    y, _ = O.attention_mixer(h, w, "l0.mix.", ATT, torch.arange(30), 1e-5)
    assert torch.allclose(trail[0], x0 + y + O.feed_forward(h, w, "l0.mlp."), atol=1e-5)


def test_oracle_layer_norm_is_torchs():
    g = torch.Generator().manual_seed(2)
    x, w, b = 5 + torch.randn(4, 24, generator=g), torch.randn(24, generator=g), torch.randn(24, generator=g)
    assert torch.allclose(O.layer_norm(x, w, b, 1e-3), torch.nn.functional.layer_norm(x, (24,), w, b, 1e-3), atol=1e-5)


def test_oracle_chunks_are_counted_from_the_start_of_the_sequence():
    ok = O.visible(torch.arange(9), torch.arange(9), 4)
    assert [r.nonzero().flatten().tolist() for r in ok] == [[0], [0, 1], [0, 1, 2], [0, 1, 2, 3], [4], [4, 5], [4, 5, 6], [4, 5, 6, 7], [8]]
    assert O.visible(torch.tensor([6]), torch.arange(9), 0)[0].nonzero().flatten().tolist() == list(range(7))


def test_oracle_sink_joins_the_denominator_only():
    s, ok = torch.tensor([[1.0, 2.0, 7.0]]), torch.tensor([[True, True, False]])
    p = O.softmax_over(s, ok, torch.tensor(0.5))
    den = math.exp(1) + math.exp(2) + math.exp(0.5)
    assert torch.allclose(p, torch.tensor([[math.exp(1) / den, math.exp(2) / den, 0.0]]))
    assert torch.allclose(O.softmax_over(s, ok).sum(), torch.tensor(1.0))


def test_oracle_rotations_pair_their_entries_and_keep_relative_angles():
    rot = {"dims": 4, "base": 100.0}
    one = torch.tensor([[[0.0, 1.0, 0.0, 0.0, 7.0, 8.0]]])
    r = O.rotate_halves(one, torch.tensor([3]), rot)[0, 0]      # entry 1 pairs with entry 3 and turns at 100^(-1/2)
    assert torch.allclose(r, torch.tensor([0.0, math.cos(0.3), 0.0, math.sin(0.3), 7.0, 8.0]), atol=1e-6)
    r = O.rotate_neighbours(one, torch.tensor([3]), rot)[0, 0]  # entry 1 pairs with entry 0 and turns at 1
    assert torch.allclose(r, torch.tensor([-math.sin(3.0), math.cos(3.0), 0.0, 0.0, 7.0, 8.0]), atol=1e-6)
    g = torch.Generator().manual_seed(4)
    q, k = torch.randn(1, 1, 6, generator=g), torch.randn(1, 1, 6, generator=g)
    for f in (O.rotate_halves, O.rotate_neighbours):
        a = (f(q, torch.tensor([9]), rot) * f(k, torch.tensor([5]), rot)).sum()
        b = (f(q, torch.tensor([14]), rot) * f(k, torch.tensor([10]), rot)).sum()
        assert torch.allclose(a, b, atol=1e-5)
        assert torch.allclose(O.rms(f(q, torch.tensor([9]), rot), 1e-3), f(O.rms(q, 1e-3), torch.tensor([9]), rot), atol=1e-6)


def test_oracle_borrowing_layer_uses_the_other_layers_keys():
    w = weights()
    pos = torch.arange(20)
    g = torch.Generator().manual_seed(5)
    h0, h3 = torch.randn(20, 24, generator=g), torch.randn(20, 24, generator=g)
    _, kv = O.attention_mixer(h0, w, "l0.mix.", ATT, pos, 1e-5)
    mx = CFG["layers"][3]["mixer"]
    y, same = O.attention_mixer(h3, w, "l3.mix.", mx, pos, 1e-5, kv)
    assert same[0] is kv[0] and same[1] is kv[1]
    full = dict(w, **{"l3.mix.k": w["l0.mix.k"], "l3.mix.v": w["l0.mix.v"]})
    k, v = O.keys_and_values(h0, full, "l3.mix.", mx, pos, 1e-5)
    assert torch.equal(k, kv[0]) and torch.equal(v, kv[1])
    assert not torch.allclose(y, O.attention_mixer(h3, full, "l3.mix.", mx, pos, 1e-5)[0], atol=1e-3)


def test_oracle_memory_decays_rows_before_the_write_and_carries_its_state():
    S0 = torch.ones(1, 2, 2)
    o, S = O.decayed_memory(torch.tensor([[[1.0, 0.0]]]), torch.tensor([[[2.0, 3.0]]]), torch.tensor([[[10.0, 20.0]]]), torch.tensor([[[0.5, 0.25]]]), S0)
    assert torch.allclose(S[0], torch.tensor([[20.5, 40.5], [30.25, 60.25]])) and torch.allclose(o[0, 0], torch.tensor([20.5, 40.5]))
    assert torch.allclose(O.channel_decay(torch.tensor([0.0]), 2.0), torch.tensor([math.sqrt(0.5)]))
    w = weights()
    h = torch.randn(19, 24, generator=torch.Generator().manual_seed(6))
    whole, _ = O.gla_mixer(h, w, "l2.mix.", GLA, 1e-5)
    a, st = O.gla_mixer(h[:8], w, "l2.mix.", GLA, 1e-5)
    b, st = O.gla_mixer(h[8:9], w, "l2.mix.", GLA, 1e-5, st)
    c, _ = O.gla_mixer(h[9:], w, "l2.mix.", GLA, 1e-5, st)
    assert torch.allclose(torch.cat([a, b, c]), whole, atol=1e-5)
