"""Host-side checks of the Zasapel model class (no GPU): the registry, the configuration reader, weight packing, and the oracle's own
mechanisms."""
import importlib
import math

import pytest
import torch

import zasapel_oracle as ref
from util import b200

F = torch.float64


def _z():
    return importlib.import_module("llm-inference-engine_b200.models.zasapel")


def test_registry_names_the_design():
    models = importlib.import_module("llm-inference-engine_b200.models")
    assert "zasapel" in models.architectures()
    assert models.architecture_of({"architecture": "Zasapel"}) == "Zasapel"


def test_layer_specs_follow_the_configuration():
    m, z = b200(), _z()
    config = ref.make_config([ref.mingru(width=21, mlp=ref.dense(ff=13)), ref.latent(heads=3, dim=10, vdim=7, kv_rank=9, q_rank=6, scale=0.5, mlp=ref.moe(experts=4, top=3, ff=5, limit=2.5)),
                              ref.latent(kv_from=1)], taps=5)
    a, b, c = z.layer_specs(config)
    assert (a["mixer"], a["norm"], a["vdim"], a["in_taps"], a["mlp"], a["expert_ff"], a["act"], a["gated"]) == (m.MIXER_MINGRU, m.NORM_RMS_SUM, 21, 5, m.MLP_DENSE, 13, m.ACT_POLYNORM, 0)
    assert (b["mixer"], b["heads"], b["dim"], b["vdim"], b["kv_rank"], b["q_rank"], b["scale"], b["head_gate"], b["kv_from"]) == (m.MIXER_LATENT, 3, 10, 7, 9, 6, 0.5, 1, -1)
    assert (b["mlp"], b["route"], b["experts"], b["top"], b["expert_ff"], b["act"], b["act_limit"], b["act_slope"], b["gated"]) == \
        (m.MLP_MOE, m.ROUTE_SIGMOID, 4, 3, 5, m.ACT_CLAMP_GLU, 2.5, 1.702, 1)
    assert c["kv_from"] == 1 and c["mlp"] == m.MLP_NONE
    assert [s["in_taps"] for s in z.layer_specs({k: v for k, v in config.items() if k != "canon"})] == [0, 0, 0]
    for bad in ({"type": "conv", "mixer": {"width": 4}, "mlp": None}, ref.latent(kv_from=0), ref.mingru(mlp={"kind": "glu"})):
        with pytest.raises(ValueError):
            z.layer_specs(ref.make_config([bad]))


def test_weights_are_packed_as_the_engine_reads_them():
    m, z = b200(), _z()
    config = ref.make_config([ref.mingru(width=6, mlp=ref.moe(experts=2, ff=4)), ref.latent(heads=2, dim=4, vdim=3, kv_rank=5, q_rank=7), ref.latent(heads=2, dim=4, vdim=3, kv_rank=5, q_rank=7, kv_from=1)],
                             width=8)
    W, packed = ref.make_weights(config, seed=1)
    specs = z.layer_specs(config)
    for i, s in enumerate(specs):
        z.fuse_layer(s, lambda n, i=i: packed[f"l{i}.{n}"], torch.float32, "cpu")
    a, b, c = specs
    assert torch.equal(a["w_in"].double(), torch.cat([W["l0.mix.z"], W["l0.mix.x"], W["l0.mix.g"]]))
    assert torch.equal(a["b_in"].double(), torch.cat([W["l0.mix.z.b"], W["l0.mix.x.b"]]))
    assert torch.equal(a["in_conv2"].double(), W["l0.canon2"].T) and torch.allclose(a["norm1"].double(), 1 + W["l0.norm1"])
    assert torch.equal(a["w_up"][1].double(), torch.cat([W["l0.mlp.e1.gate"], W["l0.mlp.e1.up"]])) and a["w_router"].shape == (2, 8)
    assert b["w_in"].shape == (7 + 5 + 2, 8) and c["w_in"].shape == (7 + 2, 8) and "kv_norm" not in c
    assert torch.equal(b["w_uk_t"][1].double(), W["l1.mix.uk"][4:].T)


def test_oracle_convolution_and_position_vector():
    x = torch.arange(12, dtype=F).view(6, 2) + 1
    w = torch.tensor([[100.0, 10.0, 1.0], [0.0, 0.0, 0.0]], dtype=F)
    out = ref.with_conv(x, w)
    assert torch.equal(out[:, 1], x[:, 1])
    assert out[0, 0] == x[0, 0] * 2 and out[1, 0] == x[1, 0] * 2 + 10 * x[0, 0] and out[4, 0] == x[4, 0] * 2 + 10 * x[3, 0] + 100 * x[2, 0]
    p = ref.position_vector(5, 7)
    assert torch.equal(p[0], torch.tensor([0.0, 1, 0, 1, 0, 1, 0], dtype=F))
    assert p[3, 0] == math.sin(3) and p[3, 1] == math.cos(3) and math.isclose(p[3, 4], math.sin(3 * 10000 ** (-4 / 7)))


def test_oracle_polynomial_of_norms_and_expert():
    z = torch.tensor([[1.0, -2.0, 3.0]], dtype=F)
    out = ref.poly_norm(z, torch.tensor([1.0, 10.0, 100.0, 7.0], dtype=F), 0.5)
    want = [v / math.sqrt(14 / 3 + 0.5) + 10 * v ** 2 / math.sqrt((1 + 16 + 81) / 3 + 0.5) + 100 * v ** 3 / math.sqrt((1 + 64 + 729) / 3 + 0.5) + 7 for v in (1.0, -2.0, 3.0)]
    assert torch.allclose(out[0], torch.tensor(want, dtype=F))
    eye = torch.eye(3, dtype=F)
    W = {"gate": eye, "up": eye.flip(0), "down": eye}
    y = ref.clamped_expert(torch.tensor([[2.0, -5.0, 0.5]], dtype=F), W, "", 1.0)
    g, u = [1.0, -5.0, 0.5], [0.5, -1.0, 1.0]
    assert torch.allclose(y[0], torch.tensor([a / (1 + math.exp(-1.702 * a)) * (b + 1) for a, b in zip(g, u)], dtype=F))


def test_oracle_weights_the_experts_input():
    config = ref.make_config([ref.mingru(mlp=ref.moe(experts=3, top=2))])
    W, _ = ref.make_weights(config, seed=2)
    ml = config["layers"][0]["mlp"]
    h = torch.randn(9, config["width"], dtype=F)
    chosen, weight = ref.route(h, W, "l0.mlp.", ml)
    assert ((weight > 0) & (weight < 1)).all() and not torch.allclose(weight.sum(-1), torch.ones(9, dtype=F))
    y = ref.feed_forward_moe(h, W, "l0.mlp.", ml)
    on_output = torch.stack([sum(w * ref.clamped_expert(h[t], W, f"l0.mlp.e{e}.", ml["expert"]["limit"]) for e, w in zip(chosen[t].tolist(), weight[t])) for t in range(9)])
    on_input = torch.stack([sum(ref.clamped_expert(w * h[t], W, f"l0.mlp.e{e}.", ml["expert"]["limit"]) for e, w in zip(chosen[t].tolist(), weight[t])) for t in range(9)])
    assert torch.allclose(y, on_input) and ref.rel_err(on_output, y) > 1e-2
