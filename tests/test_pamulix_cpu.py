"""Host-side checks of the Pamulix model class (no GPU): the registry, the configuration reader, the frequency tables, weight packing, and the
oracle's own mechanisms."""
import importlib
import math

import pytest
import torch

import pamulix_oracle as ref
from util import b200

F = torch.float64


def _p():
    return importlib.import_module("llm-inference-engine_b200.models.pamulix")


def test_registry_names_the_design():
    models = importlib.import_module("llm-inference-engine_b200.models")
    assert "pamulix" in models.architectures()


def test_layer_specs_follow_the_configuration():
    m, p = b200(), _p()
    config = ref.make_config([ref.attention(heads=6, kv_heads=3, dim=10, vdim=7, chunk=11, scale=0.5, v_mix=False, mlp=ref.moe(experts=4, top=3, ff=5)), ref.attention(), ref.latent(), ref.attention(heads=8)])
    a, b, c, d = p.layer_specs(config)
    assert (a["mixer"], a["norm"], a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["chunk"], a["scale"], a.get("v_share", 0)) == (m.MIXER_ATTN_SCORED, m.NORM_LN_POST, 6, 3, 10, 7, 11, 0.5, 0)
    assert (a["mlp"], a["route"], a["experts"], a["top"], a["expert_ff"], a["act"], a["gated"]) == (m.MLP_MOE, m.ROUTE_SOFTMAX, 4, 3, 5, m.ACT_SILU, 1)
    assert (b["v_share"], d["v_share"], b["mlp"]) == (1, 2, m.MLP_NONE)
    assert (c["mixer"], c["kv_rank"], c["q_rank"], c["rot_dim"], c["rot_dims"], c["rot_pairs"], c["head_gate"]) == (m.MIXER_LATENT, 16, 14, 8, 8, 1, 2)
    for bad in ([{"type": "conv", "mixer": dict(ref.attention()["mixer"]), "mlp": None}], [dict(ref.latent(), mlp={"kind": "dense"})], [ref.attention(), ref.attention(vdim=11)]):
        with pytest.raises(ValueError):
            p.layer_specs(ref.make_config(bad))


@pytest.mark.parametrize("kw", [{}, dict(factor=None), dict(rot_dim=32, base=50.0, factor=16.0, original=1000, fast=30.0, slow=2.0),
                                dict(rot_dim=16, base=1e6, factor=2.5, original=40, fast=1.0, slow=1.0), dict(rot_dim=2), dict(rot_dim=4, base=10.0, original=100000, fast=4.0, slow=0.5)])
def test_frequency_tables(kw):
    rot = ref.latent(**kw)["mixer"]["rot"]
    turns, amp = _p().rotation_table(rot)
    freq, want_amp = ref.pair_frequencies(rot)
    assert math.isclose(amp, want_amp) and len(turns) == rot["dims"] // 2
    assert all(math.isclose(2 * math.pi * t, f, rel_tol=1e-12) for t, f in zip(turns, freq))


def test_slowed_frequencies_by_hand():
    rot = {"base": 10000.0, "dims": 8, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}
    # pairs that make 32 and 1 turns over 2048 positions: 8 ln(2048 / 64 pi) / (2 ln 1e4) = 1.008 and 2.513: pair 1 is the last fast one, from 3 on all are slow
    freq, amp = ref.pair_frequencies(rot)
    want = [1.0, 0.1, 0.01 * (0.5 / 4 + 0.5), 0.001 / 4]
    assert all(math.isclose(a, b, rel_tol=1e-12) for a, b in zip(freq, want)) and math.isclose(amp, 1.0 + 0.1 * math.log(4.0))


def test_weights_are_packed_as_the_engine_reads_them():
    m, p = b200(), _p()
    config = ref.make_config([ref.attention(heads=2, kv_heads=1, dim=4, vdim=3, mlp=ref.moe(experts=2, ff=4)), ref.latent(heads=2, dim=4, rot_dim=2, vdim=3, kv_rank=5, q_rank=7), ref.attention(heads=2, kv_heads=1, dim=4, vdim=3)],
                             width=8)
    W, packed = ref.make_weights(config, seed=1)
    specs = p.layer_specs(config)
    for i, s in enumerate(specs):
        p.fuse_layer(s, lambda n, i=i: packed[f"l{i}.{n}"], torch.float32, "cpu")
    a, b, c = specs
    assert torch.equal(a["w_in"].double(), torch.cat([W["l0.mix.q"], W["l0.mix.k"], W["l0.mix.v"]]))
    assert a["dist_slope"].tolist() == [2.0 ** -4, 2.0 ** -8] and a["sink"].tolist() == [0.0, 0.0]
    assert "v_lambda" not in a and c["v_lambda"] == float(W["l2.mix.vmix"])
    assert torch.equal(a["w_up"][1].double(), torch.cat([W["l0.mlp.e1.gate"], W["l0.mlp.e1.up"]])) and torch.equal(a["logit_bias"].double(), W["l0.mlp.router.b"])
    assert b["w_in"].shape == (7 + 5 + 2, 8) and b["rot_turns"].dtype == torch.float64 and torch.equal(b["w_uk_t"][1].double(), W["l1.mix.uk"][4:].T)


def test_oracle_block_mask_slopes_and_extra_one():
    see = ref.chunk_mask(7, 3)
    assert see[5].tolist() == [False, False, False, True, True, True, False] and see[3].tolist() == [False] * 3 + [True] + [False] * 3
    assert [ref.slope(h, 4) for h in range(4)] == [0.25, 0.0625, 2.0 ** -6, 2.0 ** -8]
    p = ref.one_more_softmax(torch.tensor([[0.0, math.log(2.0), 5.0]], dtype=F), torch.tensor([[True, True, False]]))
    assert torch.allclose(p, torch.tensor([[0.25, 0.5, 0.0]], dtype=F))
    p = ref.one_more_softmax(torch.tensor([[-1000.0]], dtype=F), torch.tensor([[True]]))   # the extra one takes everything
    assert p.item() == 0.0


def test_oracle_rotation_and_layer_norm():
    rot = {"base": 100.0, "dims": 4}
    v = torch.tensor([[1.0, 0.0, 0.0, 2.0, 7.0]] * 3, dtype=F)
    out = ref.rotate(v, rot)
    assert torch.allclose(out[2], torch.tensor([math.cos(2), math.sin(2), -2 * math.sin(0.2), 2 * math.cos(0.2), 7.0], dtype=F))
    y = ref.layer_norm(torch.tensor([[1.0, 3.0]], dtype=F), torch.tensor([2.0, 5.0], dtype=F), 3.0)
    assert torch.allclose(y, torch.tensor([[-1.0, 2.5]], dtype=F))
