"""The Lozanex design: a decoder whose layers each have one of two mixers (attention within chunks, or the
gated delta rule with one decay per head) and a mixture of experts or none. The sublayers read the residual
stream itself; an RMS norm stands behind every sublayer and behind the embedding.

This file is the design's configuration (config.json), its tensor names and shapes, and how its layers
are put together from the framework's mixers; the engine that runs it is hybrid_engine.HybridEngine."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Iterator, List, Optional, Tuple

import torch

from .hybrid_config import ConfigError
from .mixers import Attention, ExpertMlp, HeadDelta, HybridLayer, Mixer

ARCHITECTURE = "Lozanex"


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: dict
    mlp: Optional[dict]  # None: no feed-forward


@dataclass(frozen=True)
class LozanexConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: Tuple[LayerSpec, ...]

    norm_offset = 0.0  # every norm scales by its weight

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def build_layers(self, weights: Dict[str, torch.Tensor]) -> List[HybridLayer]:
        return build_layers(self, weights)

    @classmethod
    def from_dict(cls, data: dict) -> "LozanexConfig":
        layers: List[LayerSpec] = []
        for index, entry in enumerate(data["layers"]):
            mixer, mlp = dict(entry["mixer"]), entry.get("mlp")
            _check_mixer(index, entry["type"], mixer, layers)
            if mlp is not None:
                if mlp.get("kind", "moe") != "moe":
                    raise ConfigError(f"layer {index}: unknown feed-forward kind {mlp['kind']!r}")
                if not 0 < mlp["router"]["top"] <= mlp["router"]["experts"]:
                    raise ConfigError(f"layer {index}: a token uses at least one and at most all experts")
                mlp = dict(mlp)
            layers.append(LayerSpec(entry["type"], mixer, mlp))
        if not layers:
            raise ConfigError("the model has no layers")
        return cls(vocab_size=int(data["vocab"]), hidden_size=int(data["width"]),
                   norm_eps=float(data["norm"]["eps"]), layers=tuple(layers))

    def to_dict(self) -> dict:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.norm_eps},
                "layers": [{"type": layer.type, "mixer": layer.mixer, "mlp": layer.mlp} for layer in self.layers]}


def _check_mixer(index: int, kind: str, mixer: dict, earlier: List[LayerSpec]) -> None:
    if kind not in ("attention", "delta"):
        raise ConfigError(f"layer {index}: unknown mixer {kind!r}")
    if mixer["heads"] % mixer["kv_heads"]:
        raise ConfigError(f"layer {index}: heads must be a multiple of kv_heads")
    if kind == "delta":
        return
    dims = _rotation(mixer)[0]
    if dims % 2 or not 0 <= dims <= mixer["dim"]:
        raise ConfigError(f"layer {index}: the rotated dimensions must be even and at most dim")
    if mixer.get("mask") is not None and mixer["mask"]["size"] <= 0:
        raise ConfigError(f"layer {index}: a chunk holds at least one position")
    source = mixer.get("kv_from")
    if source is not None and not (
            0 <= source < index and earlier[source].type == kind and earlier[source].mixer.get("kv_from") is None and
            all(earlier[source].mixer[name] == mixer[name] for name in ("kv_heads", "dim", "vdim"))):
        raise ConfigError(f"layer {index}: kv_from must name an earlier layer that keeps keys and values of the "
                          "same heads and sizes")


def _rotation(mixer: dict) -> Tuple[int, float]:
    rot = mixer.get("rot")
    return (0, 1.0) if rot is None else (int(rot["dims"]), float(rot["base"]))


def parameter_shapes(config: LozanexConfig) -> Iterator[Tuple[str, Tuple[int, ...]]]:
    """(tensor name, shape)."""

    width = config.hidden_size
    yield "embed", (config.vocab_size, width)
    yield "embed.norm", (width,)
    for i, layer in enumerate(config.layers):
        p, m = f"l{i}.", layer.mixer
        yield p + "norm1", (width,)
        mix = p + "mix."
        if layer.type == "delta":
            qk, v, heads = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], m["heads"]
            for name, channels in (("q", qk), ("k", qk), ("v", v)):
                yield mix + name, (channels, width)
                yield mix + name + ".conv", (channels, m["conv"])
            yield from [(mix + "b", (heads, width)), (mix + "A_log", (heads,)), (mix + "norm", (m["vdim"],)),
                        (mix + "a", (heads, width)), (mix + "dt_bias", (heads,)), (mix + "g", (v, width)),
                        (mix + "o", (width, v))]
        else:
            q, k, v = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            own = m.get("kv_from") is None
            for name, rows in (("q", q),) + ((("k", k), ("v", v)) if own else ()):
                yield from [(mix + name, (rows, width)), (mix + name + ".b", (rows,))]
            yield mix + "q.norm", (q,)
            if own:
                yield mix + "k.norm", (k,)
            yield from [(mix + "o", (width, m["heads"] * m["vdim"])), (mix + "o.b", (width,))]
        if layer.mlp is not None:
            yield p + "norm2", (width,)
            mlp, router, shared = p + "mlp.", layer.mlp["router"], layer.mlp.get("shared")
            yield mlp + "router", (router["experts"], width)
            parts = [(f"e{e}.", layer.mlp["expert"]["ff"]) for e in range(router["experts"])]
            for part, ff in parts + ([] if shared is None else [("shared.", shared["ff"])]):
                yield from [(mlp + part + "gate", (ff, width)), (mlp + part + "up", (ff, width)),
                            (mlp + part + "down", (width, ff))]
    yield "final.norm", (width,)
    yield "head", (config.vocab_size, width)


def make_weights(config: LozanexConfig, *, seed: int = 0, dtype: torch.dtype = torch.float32,
                 device: str | torch.device = "cpu") -> Dict[str, torch.Tensor]:
    """Random weights of a scale at which every mechanism matters (tests and benchmarks)."""

    generator = torch.Generator(device=device).manual_seed(seed)
    weights = {}
    for name, shape in parameter_shapes(config):
        value = torch.empty(shape, dtype=torch.float32, device=device).normal_(0.0, 1.0, generator=generator)
        leaf = name.rsplit(".", 1)[-1]
        if leaf.startswith("norm"):
            value = 1.0 + 0.1 * value
        elif leaf in ("A_log", "conv"):
            value = 0.5 * value
        elif leaf == "dt_bias":
            value = value - 2.0
        elif leaf == "b" and len(shape) == 1:
            value = 0.3 * value
        elif leaf == "router":
            value = 2.0 * value * shape[-1] ** -0.5
        elif leaf != "embed":
            value = value * shape[-1] ** -0.5
        weights[name] = value.to(dtype)
    return weights


def check_weights(config: LozanexConfig, weights: Dict[str, torch.Tensor]) -> None:
    for name, shape in parameter_shapes(config):
        if name not in weights:
            raise ConfigError(f"tensor {name} is missing")
        if tuple(weights[name].shape) != shape:
            raise ConfigError(f"tensor {name} has shape {tuple(weights[name].shape)}, expected {shape}")


def build_layers(config: LozanexConfig, weights: Dict[str, torch.Tensor]) -> List[HybridLayer]:
    """The layers with their weights packed, on the weights' device and in their dtype."""

    check_weights(config, weights)
    width, eps = config.hidden_size, config.norm_eps
    layers = []
    for i, spec in enumerate(config.layers):
        p, m = f"l{i}.", spec.mixer
        own = {name[len(p) + 4:]: value for name, value in weights.items() if name.startswith(p + "mix.")}
        sizes = dict(width=width, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], epsilon=eps)
        if spec.type == "delta":
            mixer: Mixer = HeadDelta(own, **sizes)
        else:
            dims, base = _rotation(m)
            mixer = Attention(own, **sizes, scale=m["scale"], rot_dims=dims, rot_base=base,
                              chunk=None if m.get("mask") is None else m["mask"]["size"], kv_from=m.get("kv_from"))
        layer = HybridLayer(mixer, None, weights[p + "norm1"])
        if spec.mlp is not None:
            part = lambda prefix: {name: weights[f"{p}mlp.{prefix}.{name}"] for name in ("gate", "up", "down")}
            shared = None if spec.mlp.get("shared") is None else part("shared")
            layer.mlp = ExpertMlp(weights[p + "mlp.router"], [part(f"e{e}") for e in range(spec.mlp["router"]["experts"])],
                                  width=width, top=spec.mlp["router"]["top"], shared=shared)
            layer.mlp_norm_out = weights[p + "norm2"]
        layers.append(layer)
    return layers
