"""Manapel: a small decoder-only language model with a tanh norm before and after every sublayer,

    x <- x + norm_b(sublayer(norm_a(x))),   norm(z) = tanh(alpha z) * w + b

(alpha one number, w and b vectors; no mean and no variance anywhere). The mixer is grouped-query attention over everything
before, with biased projections, rotary positions in halves and every rotated query / key head divided by its root mean
square; a layer may read the keys and values of an earlier layer instead of having its own (`kv_from`). The feed-forward is a
ReLU-gated unit or a mixture of squared-ReLU experts (largest router logits, softmax over the chosen ones) with a shared
expert that every token uses. The head is a matrix of its own, logits are scaled. The reference has no such model; it is
served the way the other native decoders are: configuration and weights from a checkpoint folder (config.json +
model.safetensors), the CUDA engine (llark_b200.engine_manapel), the slot cache (llark_b200.state_cache), `generate()`
through llark_b200.generate and batches through llark_b200.scheduler.

config.json keys: architecture ("Manapel"), vocab, width, norm.eps (of the heads' root mean square), logit_scale, layers[]
with type ("attention"), mixer {...}, mlp (null | {kind: "dense", ff} | {kind: "moe", expert.ff, router {experts, top},
shared (null | {ff})}).
  attention:  heads, kv_heads, dim, vdim, scale, rot {base, dims}, kv_from (optional: number of an earlier layer with keys
              and values of its own);  tensors q, k, v (+ .b each), o; without k and v when kv_from is given
Other tensors: embed, head, final.norm, l<i>.norm1 / norm1b / norm2 / norm2b (each with .alpha and .b), l<i>.mlp.gate / up /
down (dense), l<i>.mlp.router (+ .b), l<i>.mlp.e<j>.up / down, l<i>.mlp.shared.up / down (moe).
"""
from dataclasses import dataclass, field
from typing import List, Optional

from llark_b200.models.native import NativeCausalLM

ARCHITECTURE = "Manapel"
# the configuration's layer types and feed-forward kinds -> entries of llark_b200.mixers.MIXERS / FEED_FORWARDS
MIXER_TYPES = {"attention": "rotary_attention_unit"}
FEED_FORWARD_KINDS = {"dense": "relu_glu", "moe": "moe_top_softmax"}
SHARED_SIZES = ("kv_heads", "dim", "vdim", "rot")  # what a layer and the one it reads keys and values from agree on


@dataclass
class ManapelLayer:
    type: str
    mixer: dict
    mlp: Optional[dict] = None


@dataclass
class ManapelConfig:
    vocab: int
    width: int
    eps: float
    logit_scale: float = 1.0
    layers: List[ManapelLayer] = field(default_factory=list)
    eos_token_id: Optional[int] = None
    pad_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, d):
        from llark_b200.mixers import FEED_FORWARDS, MIXERS

        if d.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} configuration: architecture = {d.get('architecture')!r}")
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] not in MIXER_TYPES or MIXER_TYPES[e["type"]] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r} (known: {sorted(MIXER_TYPES)})")
            mixer, mlp = dict(e["mixer"]), e.get("mlp")
            j = mixer.get("kv_from")
            if j is not None:
                if not 0 <= int(j) < i:
                    raise ValueError(f"layer {i}: kv_from must name an earlier layer")
                other = layers[int(j)].mixer
                if other.get("kv_from") is not None:
                    raise ValueError(f"layer {i}: layer {j} has no keys and values of its own")
                if any(mixer.get(k) != other.get(k) for k in SHARED_SIZES):
                    raise ValueError(f"layer {i}: {', '.join(SHARED_SIZES)} must equal those of layer {j}")
            if mlp is not None and (mlp.get("kind") not in FEED_FORWARD_KINDS
                                    or FEED_FORWARD_KINDS[mlp["kind"]] not in FEED_FORWARDS):
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r} (known: {sorted(FEED_FORWARD_KINDS)})")
            layers.append(ManapelLayer(type=e["type"], mixer=mixer, mlp=dict(mlp) if mlp else None))
        if not layers:
            raise ValueError("a model needs at least one layer")
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]),
                   logit_scale=float(d.get("logit_scale", 1.0)), layers=layers, eos_token_id=d.get("eos_token_id"),
                   pad_token_id=d.get("pad_token_id"))

    def to_dict(self):
        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "logit_scale": self.logit_scale,
                "layers": [{"type": l.type, "mixer": l.mixer, "mlp": l.mlp} for l in self.layers]}


class ManapelForCausalLM(NativeCausalLM):
    """Inference-only model object: configuration + engine (llark_b200.models.native.NativeCausalLM)."""
    config_class = ManapelConfig

    @staticmethod
    def engine_class():
        from llark_b200.engine_manapel import ManapelEngine

        return ManapelEngine
