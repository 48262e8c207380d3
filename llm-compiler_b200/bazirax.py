"""The Bazirax design: a decoder whose layers each have one of three mixers (retention, latent attention,
gated delta rule), a gated MLP or none, and an RMS norm before and after every sublayer.

This file is the design's configuration (config.json), its tensor names and shapes, and how its layers
are put together from the framework's mixers; the engine that runs it is hybrid_engine.HybridEngine."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Iterator, List, Optional, Tuple

import torch

from .hybrid_config import ConfigError
from .mixers import ChannelDelta, GatedMlp, HybridLayer, LatentAttention, Mixer, Retention

ARCHITECTURE = "Bazirax"


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: dict
    ff: Optional[int]  # None: no feed-forward


@dataclass(frozen=True)
class BaziraxConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: Tuple[LayerSpec, ...]

    norm_offset = 1.0  # the residual norms scale by 1 + their weight

    def build_layers(self, weights: Dict[str, torch.Tensor]) -> List[HybridLayer]:
        return build_layers(self, weights)

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, data: dict) -> "BaziraxConfig":
        layers = []
        for index, entry in enumerate(data["layers"]):
            mixer = dict(entry["mixer"])
            _check_mixer(index, entry["type"], mixer, layers)
            mlp = entry.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ConfigError(f"layer {index}: unknown feed-forward kind {mlp['kind']!r}")
            layers.append(LayerSpec(entry["type"], mixer, None if mlp is None else int(mlp["ff"])))
        if not layers:
            raise ConfigError("the model has no layers")
        return cls(vocab_size=int(data["vocab"]), hidden_size=int(data["width"]),
                   norm_eps=float(data["norm"]["eps"]), layers=tuple(layers))

    def to_dict(self) -> dict:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.norm_eps},
                "layers": [{"type": layer.type, "mixer": layer.mixer,
                            "mlp": None if layer.ff is None else {"kind": "dense", "ff": layer.ff}}
                           for layer in self.layers]}


def _check_mixer(index: int, kind: str, mixer: dict, earlier: List[LayerSpec]) -> None:
    if kind == "retention":
        if len(mixer["decay"]) != mixer["heads"]:
            raise ConfigError(f"layer {index}: one decay per head is needed")
        dims = mixer["rot"]["dims"]
        if dims % 2 or not 0 <= dims <= mixer["dim"]:
            raise ConfigError(f"layer {index}: the rotated dimensions must be even and at most dim")
    elif kind == "channel_delta":
        if mixer["heads"] % mixer["kv_heads"]:
            raise ConfigError(f"layer {index}: heads must be a multiple of kv_heads")
    elif kind == "latent_attention":
        source = mixer.get("kv_from")
        if source is not None and not (0 <= source < index and earlier[source].type == kind and
                                       earlier[source].mixer.get("kv_from") is None and
                                       earlier[source].mixer["kv_rank"] == mixer["kv_rank"]):
            raise ConfigError(f"layer {index}: kv_from must name an earlier layer that keeps latents of the "
                              "same rank")
    else:
        raise ConfigError(f"layer {index}: unknown mixer {kind!r}")


def parameter_shapes(config: BaziraxConfig, *, gate_rank: int = 16) -> Iterator[Tuple[str, Tuple[int, ...]]]:
    """(tensor name, shape). The rank of the delta rule's two low-rank projections is a property of the
    weights (their shapes), not of config.json: `gate_rank`."""

    width = config.hidden_size
    yield "embed", (config.vocab_size, width)
    for i, layer in enumerate(config.layers):
        p, m = f"l{i}.", layer.mixer
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if layer.ff is not None else ()):
            yield p + name, (width,)
        mix = p + "mix."
        if layer.type == "retention":
            qk, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            yield from [(mix + "q", (qk, width)), (mix + "k", (qk, width)), (mix + "v", (v, width)),
                        (mix + "g", (v, width)), (mix + "o", (width, v))]
        elif layer.type == "channel_delta":
            qk, decay, v = m["kv_heads"] * m["dim"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for name, channels in (("q", qk), ("k", qk), ("v", v)):
                yield mix + name, (channels, width)
                yield mix + name + ".conv", (channels, m["conv"])
            yield from [(mix + "b", (m["heads"], width)), (mix + "A_log", (m["heads"],)),
                        (mix + "norm", (m["vdim"],)), (mix + "a1", (gate_rank, width)),
                        (mix + "a2", (decay, gate_rank)), (mix + "dt_bias", (decay,)),
                        (mix + "g1", (gate_rank, width)), (mix + "g2", (v, gate_rank)),
                        (mix + "o", (width, v))]
        else:
            qk, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            yield from [(mix + "dq", (m["q_rank"], width)), (mix + "dq.norm", (m["q_rank"],)),
                        (mix + "uq", (qk, m["q_rank"]))]
            if m.get("kv_from") is None:
                yield from [(mix + "dkv", (m["kv_rank"], width)), (mix + "dkv.norm", (m["kv_rank"],))]
            yield from [(mix + "uk", (qk, m["kv_rank"])), (mix + "uv", (v, m["kv_rank"])),
                        (mix + "sink", (m["heads"],)), (mix + "o", (width, v))]
        if layer.ff is not None:
            mlp = p + "mlp."
            yield from [(mlp + "gate", (layer.ff, width)), (mlp + "up", (layer.ff, width)),
                        (mlp + "down", (width, layer.ff))]
    yield "final.norm", (width,)
    yield "head", (config.vocab_size, width)


def make_weights(config: BaziraxConfig, *, seed: int = 0, dtype: torch.dtype = torch.float32,
                 device: str | torch.device = "cpu", gate_rank: int = 16) -> Dict[str, torch.Tensor]:
    """Random weights of a scale at which every mechanism matters (tests and benchmarks)."""

    generator = torch.Generator(device=device).manual_seed(seed)
    weights = {}
    for name, shape in parameter_shapes(config, gate_rank=gate_rank):
        value = torch.empty(shape, dtype=torch.float32, device=device).normal_(0.0, 1.0, generator=generator)
        leaf = name.rsplit(".", 1)[-1]
        if name.endswith(("dq.norm", "dkv.norm", "mix.norm")):
            value = 1.0 + 0.1 * value
        elif leaf.startswith("norm"):
            value = 0.1 * value
        elif leaf == "A_log":
            value = 0.5 * value
        elif leaf == "dt_bias":
            value = value - 2.0
        elif leaf == "conv":
            value = 0.5 * value
        elif leaf not in ("embed", "sink"):
            value = value * shape[-1] ** -0.5
        weights[name] = value.to(dtype)
    return weights


def check_weights(config: BaziraxConfig, weights: Dict[str, torch.Tensor]) -> None:
    ranks = {name: weights[name].shape[0] for name in weights if name.endswith((".mix.a1", ".mix.g1"))}
    for name, shape in parameter_shapes(config):
        if name not in weights:
            raise ConfigError(f"tensor {name} is missing")
        low = name[:-1] + "1"  # a2 -> a1, g2 -> g1
        if name in ranks:
            shape = (ranks[name], shape[1])
        elif name.endswith((".mix.a2", ".mix.g2")) and low in ranks:
            shape = (shape[0], ranks[low])
        if tuple(weights[name].shape) != shape:
            raise ConfigError(f"tensor {name} has shape {tuple(weights[name].shape)}, expected {shape}")


def build_layers(config: BaziraxConfig, weights: Dict[str, torch.Tensor]) -> List[HybridLayer]:
    """The layers with their weights packed, on the weights' device and in their dtype."""

    check_weights(config, weights)
    width, eps = config.hidden_size, config.norm_eps
    layers = []
    for i, spec in enumerate(config.layers):
        p, m = f"l{i}.", spec.mixer
        own = {name[len(p) + 4:]: value for name, value in weights.items() if name.startswith(p + "mix.")}
        if spec.type == "retention":
            mixer: Mixer = Retention(own, width=width, heads=m["heads"], dim=m["dim"], vdim=m["vdim"],
                                     decay=m["decay"], rot_dims=m["rot"]["dims"], rot_base=m["rot"]["base"],
                                     epsilon=eps)
        elif spec.type == "channel_delta":
            mixer = ChannelDelta(own, width=width, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"],
                                 vdim=m["vdim"], epsilon=eps)
        else:
            mixer = LatentAttention(own, width=width, heads=m["heads"], dim=m["dim"], vdim=m["vdim"],
                                    q_rank=m["q_rank"], kv_rank=m["kv_rank"], scale=m["scale"], epsilon=eps,
                                    kv_from=m.get("kv_from"))
        layer = HybridLayer(mixer, weights[p + "norm1"], weights[p + "norm1b"])
        if spec.ff is not None:
            mlp = {name: weights[p + "mlp." + name] for name in ("gate", "up", "down")}
            layer.mlp = GatedMlp(mlp, width=width)
            layer.mlp_norm_in, layer.mlp_norm_out = weights[p + "norm2"], weights[p + "norm2b"]
        layers.append(layer)
    return layers
