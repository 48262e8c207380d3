"""Host side of the hybrid designs: configuration, weight files, packing, slots, scheduling, and the plain
implementation the GPU tests compare with (its own invariants)."""

import json
import struct

import pytest
import torch

from llm_compiler_b200 import bazirax, mixers, registry
from llm_compiler_b200.kv_state import ExecutionError, SlotState
from llm_compiler_b200.safetensors_io import load_safetensors, save_safetensors
from llm_compiler_b200.scheduler import RequestScheduler
from oracle import hybrid_model as oracle


def tiny():
    return {"architecture": "Bazirax", "vocab": 24, "width": 20, "norm": {"eps": 1e-4}, "layers": [
        {"type": "retention", "mlp": None, "mixer": {"heads": 2, "dim": 6, "vdim": 5, "decay": [0.9, 0.5],
                                                     "rot": {"base": 100.0, "dims": 4}}},
        {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 12},
         "mixer": {"heads": 3, "dim": 4, "vdim": 6, "q_rank": 7, "kv_rank": 5, "scale": 0.5}},
        {"type": "channel_delta", "mlp": {"kind": "dense", "ff": 9},
         "mixer": {"heads": 4, "kv_heads": 2, "dim": 3, "vdim": 5, "conv": 2}},
        {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 12},
         "mixer": {"heads": 2, "dim": 5, "vdim": 3, "q_rank": 4, "kv_rank": 5, "scale": 0.4, "kv_from": 1}}]}


def test_configuration_round_trip_and_registry():
    entry = registry.entry_of(tiny())
    config = entry.read_config(tiny())
    assert config.to_dict() == tiny()
    assert entry.portions and {"Bazirax", "Qwen2ForCausalLM"} <= set(registry.architectures())
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.entry_of({"architecture": "none such"})


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0]["mixer"]["decay"].append(0.1),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3),
    lambda c: c["layers"][2]["mixer"].update(kv_heads=3),
    lambda c: c["layers"][3]["mixer"].update(kv_from=0),
    lambda c: c["layers"][3]["mixer"].update(kv_from=3),
    lambda c: c["layers"][3]["mixer"].update(kv_rank=6),
    lambda c: c["layers"][1].update(type="other"),
    lambda c: c["layers"][1].update(mlp={"kind": "sparse", "ff": 3}),
    lambda c: c.update(layers=[]),
])
def test_contradictory_configurations_are_refused(change):
    config = tiny()
    change(config)
    with pytest.raises(bazirax.ConfigError):
        bazirax.BaziraxConfig.from_dict(config)


def test_weights_are_checked_against_the_configuration():
    config = bazirax.BaziraxConfig.from_dict(tiny())
    weights = bazirax.make_weights(config, gate_rank=3)
    bazirax.check_weights(config, weights)
    missing = dict(weights)
    del missing["l3.mix.uk"]
    with pytest.raises(bazirax.ConfigError, match="missing"):
        bazirax.check_weights(config, missing)
    with pytest.raises(bazirax.ConfigError, match="shape"):
        bazirax.check_weights(config, dict(weights, head=torch.zeros(24, 19)))
    with pytest.raises(bazirax.ConfigError, match="shape"):
        bazirax.check_weights(config, {**weights, "l2.mix.a2": torch.zeros(12, 4)})
    assert "l3.mix.dkv" not in weights and "l0.norm2" not in weights
    layers = bazirax.build_layers(config, weights)
    assert layers[0].mlp is None and layers[3].mixer.shared_state == 1
    assert layers[3].mixer.state_spec(10) == {}


def test_packed_projections_are_the_projections():
    config = bazirax.BaziraxConfig.from_dict(tiny())
    weights = bazirax.make_weights(config, gate_rank=3)
    delta = bazirax.build_layers(config, weights)[2].mixer
    h = torch.randn(4, 20)
    padded = torch.zeros(4, 24)
    padded[:, :20] = h
    projected = padded @ delta.w_in.T
    for column, name in zip(delta.columns, ("q", "k", "v", "b")):
        w = weights["l2.mix." + name]
        assert column % 8 == 0
        assert torch.allclose(projected[:, column:column + w.shape[0]], h @ w.T, atol=1e-5)
    gates = projected[:, delta.low_column:] @ delta.w_gates.T
    for column, (low, up) in ((delta.decay_column, ("a1", "a2")), (delta.gate_column, ("g1", "g2"))):
        want = (h @ weights["l2.mix." + low].T) @ weights["l2.mix." + up].T
        assert torch.allclose(gates[:, column:column + want.shape[1]], want, atol=1e-5)
    assert mixers.pad_heads(torch.ones(6, 2), 3, 4).tolist()[2:4] == [[0, 0], [0, 0]]


def test_safetensors_round_trip_and_refusals(tmp_path):
    tensors = {"a": torch.randn(3, 5).to(torch.bfloat16), "b": torch.arange(7, dtype=torch.int32),
               "c": torch.tensor(2.5), "d": torch.zeros(0, 4)}
    path = tmp_path / "model.safetensors"
    save_safetensors(tensors, path)
    loaded = load_safetensors(path)
    assert list(loaded) == list(tensors)
    for name, tensor in tensors.items():
        assert loaded[name].dtype == tensor.dtype and torch.equal(loaded[name], tensor)
    data = path.read_bytes()
    header = {"a": {"dtype": "F32", "shape": [4], "data_offsets": [0, 12]}}
    text = json.dumps(header).encode()
    path.write_bytes(struct.pack("<Q", len(text)) + text + bytes(16))
    with pytest.raises(ValueError, match="does not lie inside"):
        load_safetensors(path)
    path.write_bytes(data[:4])
    with pytest.raises(ValueError):
        load_safetensors(path)


def test_slots_are_handed_out_lowest_first_and_counted():
    state = SlotState([{"x": ((2,), torch.float32)}, {}], slots=3, capacity=8, device="cpu")
    assert [state.acquire() for _ in range(3)] == [0, 1, 2]
    with pytest.raises(ExecutionError):
        state.acquire()
    state.host_lengths[1] = 5
    with pytest.raises(ExecutionError):
        state.require(1, 4)
    state.require(1, 3)
    state.release(1)
    with pytest.raises(ExecutionError):
        state.release(1)
    assert state.acquire() == 1 and state.host_lengths[1] == 0
    assert state.bytes() == 3 * 2 * 4 and state.slots_in_use() == 3


class CountingEngine:
    """A stand-in engine whose next token is (last token + tokens seen) mod 97."""

    def __init__(self, batch, capacity):
        self.batch, self.capacity = batch, capacity
        self.state = SlotState([], slots=batch, capacity=capacity, device="cpu")
        self.state.check = lambda: None
        self.seen = {}
        self.widest = 0

    def open(self):
        slot = self.state.acquire()
        self.seen[slot] = 0
        return slot

    def close(self, slot):
        self.state.release(slot)

    def decode_rows(self, slots, tokens, *, use_graph=True):
        self.widest = max(self.widest, len(slots))
        out = []
        for slot, token in zip(slots, tokens):
            self.seen[slot] += 1
            out.append((token + self.seen[slot]) % 97)
        return out

    def forward(self, entries, want):
        rows = []
        for (slot, tokens), places in zip(entries, want):
            self.seen[slot] += len(tokens)
            rows += [(tokens[-1] + self.seen[slot]) % 97 for _ in places]
        self.last = rows
        return torch.nn.functional.one_hot(torch.tensor(rows), 97).float() if rows else None


def test_scheduler_batches_portions_and_decoding(monkeypatch):
    from llm_compiler_b200 import scheduler as module

    monkeypatch.setattr(module.kernels, "b200_argmax", lambda logits: logits.argmax(-1))
    engine = CountingEngine(batch=3, capacity=64)
    scheduler = RequestScheduler(engine, max_portion=8)
    prompts = [[5] * 20, [1, 2, 3], [9], [4] * 11, [7, 7]]
    requests = [scheduler.submit(p, n) for p, n in zip(prompts, (4, 6, 1, 3, 5))]
    scheduler.run()
    for request, prompt in zip(requests, prompts):
        token, seen, want = prompt[-1], len(prompt), []
        for _ in range(request.max_new_tokens):
            token = (token + seen) % 97
            want.append(token)
            seen += 1
        assert request.output == want
    assert engine.state.slots_in_use() == 0 and engine.widest >= 2
    stopped = scheduler.submit([3], 9, stop_token=4)  # 3 + 1
    scheduler.run()
    assert stopped.output == [4]
    with pytest.raises(ExecutionError):
        scheduler.submit([1] * 60, 6)
    with pytest.raises(ValueError):
        scheduler.submit([], 3)


# ------------------------------------------------------- the plain implementation itself ----
def test_oracle_mechanisms_against_closed_forms():
    x = torch.randn(4, 2, 6, dtype=torch.float64)
    turned = oracle.rotate_half(x, 50.0, 4, first=3)
    assert torch.allclose(turned.norm(dim=-1), x.norm(dim=-1)) and torch.equal(turned[..., 4:], x[..., 4:])
    conv = oracle.causal_conv(torch.eye(3, dtype=torch.float64)[:, :1], torch.tensor([[3.0, 2.0, 1.0]]))
    assert conv[:, 0].tolist() == [1.0, 2.0, 3.0]  # last tap: the current token
    q = k = torch.ones(3, 1, 1, dtype=torch.float64)
    v = torch.tensor([1.0, 2.0, 4.0], dtype=torch.float64).view(3, 1, 1)
    assert oracle.retention_scan(q, k, v, [0.5]).flatten().tolist() == [1.0, 2.5, 5.25]
    one = torch.ones(3, 1, 1, dtype=torch.float64)
    full = oracle.delta_scan(q, k, v, one, torch.ones(3, 1, dtype=torch.float64))
    assert full.flatten().tolist() == [1.0, 2.0, 4.0]  # beta 1 on a unit key: the old value is replaced
    half = oracle.delta_scan(q, k, v, one, torch.full((3, 1), 0.5, dtype=torch.float64))
    assert half.flatten().tolist() == [0.5, 1.25, 2.625]
    sink = torch.zeros(1, dtype=torch.float64)
    out = oracle.sink_attention(torch.zeros_like(q), k, one, 1.0, sink)
    assert torch.allclose(out.flatten(), torch.tensor([1 / 2, 2 / 3, 3 / 4], dtype=torch.float64))


def test_oracle_is_causal_and_a_planted_mistake_shows():
    config = tiny()
    weights = bazirax.make_weights(bazirax.BaziraxConfig.from_dict(config), gate_rank=3)
    tokens = list(range(12))
    full = oracle.forward(config, weights, tokens)
    assert torch.allclose(oracle.forward(config, weights, tokens[:7]), full[:7])
    for change in (lambda c: c["layers"][0]["mixer"].update(decay=[0.9, 0.52]),
                   lambda c: c["layers"][1]["mixer"].update(scale=0.55),
                   lambda c: c["layers"][0]["mixer"]["rot"].update(base=110.0)):
        wrong = tiny()
        change(wrong)
        assert float((oracle.forward(wrong, weights, tokens) - full).abs().max()) > 1e-4
    without_sink = {n: torch.full_like(w, -1e4) if n.endswith("sink") else w for n, w in weights.items()}
    assert float((oracle.forward(config, without_sink, tokens) - full).abs().max()) > 1e-3
