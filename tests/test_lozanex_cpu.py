"""Host side of the Lozanex design: configuration, tensor names, packing, and the invariants of the plain
implementation that the GPU tests compare with."""

import copy

import pytest
import torch

from llm_compiler_b200 import lozanex, registry
from llm_compiler_b200.hybrid_config import ConfigError
from oracle import hybrid_model as oracle


def tiny():
    moe = {"kind": "moe", "expert": {"ff": 7}, "router": {"experts": 4, "top": 2}, "shared": {"ff": 10}}
    attention = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 5, "scale": 0.4, "rot": {"base": 100.0, "dims": 4},
                 "mask": {"size": 5}}
    return {"architecture": "Lozanex", "vocab": 24, "width": 20, "norm": {"eps": 1e-4}, "layers": [
        {"type": "delta", "mlp": moe, "mixer": {"heads": 4, "kv_heads": 2, "dim": 3, "vdim": 5, "conv": 2}},
        {"type": "attention", "mlp": None, "mixer": attention},
        {"type": "attention", "mlp": {**moe, "router": {"experts": 3, "top": 1}},
         "mixer": {**attention, "scale": 0.3, "mask": {"size": 4}, "kv_from": 1}}]}


def test_configuration_round_trip_and_registry():
    entry = registry.entry_of(tiny())
    config = entry.read_config(tiny())
    assert config.to_dict() == tiny() and entry.portions
    assert {"Bazirax", "Lozanex", "Qwen2ForCausalLM"} <= set(registry.architectures())


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mixer"].update(kv_heads=3),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=3),
    lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][2]["mixer"].update(kv_from=0),
    lambda c: c["layers"][2]["mixer"].update(kv_from=2),
    lambda c: c["layers"][2]["mixer"].update(vdim=6),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=5),
    lambda c: c["layers"][0]["mlp"].update(kind="dense"),
    lambda c: c.update(layers=[]),
])
def test_contradictory_configurations_are_refused(change):
    config = copy.deepcopy(tiny())
    change(config)
    with pytest.raises(ConfigError):
        lozanex.LozanexConfig.from_dict(config)


def test_weights_are_checked_and_packed():
    config = lozanex.LozanexConfig.from_dict(tiny())
    weights = lozanex.make_weights(config)
    missing = dict(weights)
    del missing["l0.mlp.e3.up"]
    with pytest.raises(ConfigError, match="missing"):
        lozanex.check_weights(config, missing)
    with pytest.raises(ConfigError, match="shape"):
        lozanex.check_weights(config, {**weights, "l1.mix.q.norm": torch.zeros(6)})
    assert "l2.mix.k" not in weights and "l1.norm2" not in weights
    layers = lozanex.build_layers(config, weights)
    assert layers[1].mlp is None and layers[2].mixer.shared_state == 1 and layers[2].mixer.state_spec(9) == {}
    assert all(layer.norm_in is None for layer in layers)
    h = torch.randn(4, 20)
    rows = torch.zeros(4, 24)
    rows[:, :20] = h
    attention = layers[1].mixer
    projected = rows @ attention.w_in.T + attention.bias
    for column, name in zip(attention.columns, ("q", "k", "v")):
        want = h @ weights["l1.mix." + name].T + weights["l1.mix." + name + ".b"]
        assert column % 8 == 0 and torch.allclose(projected[:, column:column + want.shape[1]], want, atol=1e-5)
    delta = layers[0].mixer
    projected = rows @ delta.w_in.T
    for column, name in zip((*delta.columns, delta.decay_column, delta.gate_column), "qkvbag"):
        want = h @ weights["l0.mix." + name].T
        assert torch.allclose(projected[:, column:column + want.shape[1]], want, atol=1e-5)
    experts = layers[0].mlp
    inner = torch.einsum("nk,rk->rn", experts.w_in[2], rows)
    mixed = oracle.silu(inner[:, 0::2]) * inner[:, 1::2]
    want = oracle.dense_mlp({name: weights["l0.mlp.e2." + name] for name in ("gate", "up", "down")}, h)
    assert torch.allclose((mixed @ experts.w_out[2].T)[:, :20], want, atol=1e-4)
    assert [experts.tile_of(rows) for rows in (1, 64, 65, 128, 129, 5000)] == [64, 64, 128, 128, 128, 256]
    # the shared expert in slices of the others' size: their sum is the whole
    assert experts.slices == 2 and experts.w_in.shape[0] == 6
    parts = [((oracle.silu(inner[:, 0::2]) * inner[:, 1::2]) @ experts.w_out[e].T)[:, :20]
             for e in (4, 5) for inner in (rows @ experts.w_in[e].T,)]
    shared = {name: weights["l0.mlp.shared." + name] for name in ("gate", "up", "down")}
    assert torch.allclose(sum(parts), oracle.dense_mlp(shared, h), atol=1e-4)
    inner = rows @ experts.shared.w_in.T
    dense = (oracle.silu(inner[:, 0::2]) * inner[:, 1::2]) @ experts.shared.w_out.T
    assert torch.allclose(dense[:, :20], oracle.dense_mlp(shared, h), atol=1e-4)


# ------------------------------------------------------- the plain implementation itself ----
def test_oracle_mechanisms_against_closed_forms():
    one = torch.ones(6, 1, 1, dtype=torch.float64)
    v = torch.arange(6, dtype=torch.float64).view(6, 1, 1)
    # equal scores: the mean of the chunk's values so far
    assert oracle.chunk_attention(0 * one, one, v, 1.0, 4).flatten().tolist() == [0.0, 0.5, 1.0, 1.5, 4.0, 4.5]
    assert oracle.chunk_attention(0 * one, one, v, 1.0, None).flatten().tolist() == [0.0, 0.5, 1.0, 1.5, 2.0, 2.5]
    heads = oracle.chunk_attention(torch.zeros(2, 4, 1), torch.ones(2, 2, 1), torch.tensor([[[1.0], [2.0]]] * 2), 1.0, 2)
    assert heads[1].flatten().tolist() == [1.0, 1.0, 2.0, 2.0]  # neighbouring query heads share a key head
    scores, chosen = oracle.route(torch.eye(3, dtype=torch.float64), torch.tensor([[0.0, 2.0, -1.0]], dtype=torch.float64), 2)
    assert chosen.tolist() == [[1, 0]] and abs(float(scores[0, 1]) - 0.5) < 1e-12
    w = {"router": torch.tensor([[0.0]]), **{f"{part}.{name}": torch.ones(1, 1) for part in ("e0", "shared")
                                             for name in ("gate", "up", "down")}}
    spec = {"router": {"top": 1}, "shared": {"ff": 1}}
    silu = lambda z: z / (1 + torch.exp(-z))
    z = torch.tensor([[2.0]])
    assert torch.allclose(oracle.expert_mlp(w, spec, z), silu(0.5 * z) * 0.5 * z + silu(z) * z)  # score 1/2 on the input


def test_oracle_is_causal_and_a_planted_mistake_shows():
    config = tiny()
    weights = lozanex.make_weights(lozanex.LozanexConfig.from_dict(config))
    tokens = list(range(13))
    full = oracle.lozanex_forward(config, weights, tokens)
    assert torch.allclose(oracle.lozanex_forward(config, weights, tokens[:7]), full[:7])
    for change in (lambda c: c["layers"][1]["mixer"]["mask"].update(size=6),
                   lambda c: c["layers"][2]["mixer"]["mask"].update(size=3),
                   lambda c: c["layers"][2]["mixer"].update(scale=0.35),
                   lambda c: c["layers"][1]["mixer"]["rot"].update(base=110.0),
                   lambda c: c["layers"][0]["mlp"]["router"].update(top=1)):
        wrong = copy.deepcopy(config)
        change(wrong)
        assert float((oracle.lozanex_forward(wrong, weights, tokens) - full).abs().max()) > 1e-4
    for name in ("l1.mix.q.b", "l1.mix.o.b", "l0.mix.dt_bias", "l0.mix.A_log"):
        changed = {**weights, name: weights[name] + 0.2}
        assert float((oracle.lozanex_forward(config, changed, tokens) - full).abs().max()) > 1e-4
