"""Family registry: static descriptors that detect a checkpoint's family, open it into a typed
model description, classify every tensor into a component role, and say which stored formats the
engine has kernels for.  An unsupported operand is a *result* (a ``Hint`` saying what is missing
and what would fix it), never an exception.

Counterpart: rust/crates/cuteafd-loader/src/plan/family.rs:19-256 (Hint, ExpertContract,
FamilyModel, Family, REGISTRY, detect) and plan/spec.rs (Component roles).
"""
from __future__ import annotations

import re
from dataclasses import dataclass, field

from ..config import ModelConfig
from .formats import QuantOperand

ROLES = ("embedding", "head", "final_norm", "norm", "attention", "indexer", "router", "routed_expert",
         "shared_expert", "dense_ffn", "mtp", "other")


@dataclass(frozen=True)
class Hint:
    what: str      # what cannot be served as stored
    how: str       # what would make it servable


@dataclass
class ExpertContract:
    """What the expert ranks of this family must provide."""
    activation: str = "silu"
    formats: tuple[str, ...] = ("bf16", "fp8_block128", "nvfp4", "mxfp4", "exl3")
    wire: str = "bf16"
    slice_granule: int = 128


@dataclass
class FamilyModel:
    family: "Family"
    cfg: ModelConfig
    contract: ExpertContract = field(default_factory=ExpertContract)

    _LAYER = re.compile(r"model\.layers\.(\d+)\.(.*)")

    def classify(self, name: str) -> tuple[str, int | None, int | None]:
        """(role, layer, expert) of a tensor name."""
        if name.startswith("model.embed_tokens"):
            return "embedding", None, None
        if name.startswith("lm_head"):
            return "head", None, None
        if name.startswith("model.norm"):
            return "final_norm", None, None
        m = self._LAYER.match(name)
        if not m:
            return "other", None, None
        layer, rest = int(m.group(1)), m.group(2)
        if layer >= self.cfg.num_layers and not rest.startswith("mlp.experts"):
            return "mtp", layer, None
        if "indexer" in rest:
            return "indexer", layer, None
        if rest.startswith("self_attn"):
            return "attention", layer, None
        if rest.startswith("mlp.experts."):
            return "routed_expert", layer, int(rest.split(".")[2])
        if rest.startswith("mlp.shared_expert"):
            return "shared_expert", layer, None
        if rest.startswith("mlp.gate.") :
            return "router", layer, None
        if rest.startswith("mlp."):
            return "dense_ffn", layer, None
        if "norm" in rest:
            return "norm", layer, None
        return "other", layer, None

    def accepts(self, op: QuantOperand, role: str) -> Hint | None:
        """None when the engine serves this operand as stored; otherwise the reason."""
        fmt = op.format.split("_k")[0] if op.format.startswith("exl3") else op.format
        if role in ("embedding", "head", "final_norm", "norm", "router"):
            if op.encoding not in ("bf16", "f16", "f32"):
                return Hint(f"{op.name}: {role} stored as {op.format}", "store norms, router, embedding and head in bf16/f32")
            return None
        if role == "routed_expert":
            if fmt not in self.contract.formats:
                return Hint(f"{op.name}: routed expert stored as {op.format}",
                            f"supported expert formats: {', '.join(self.contract.formats)}")
            if op.shape[1] % 128 and fmt != "bf16":
                return Hint(f"{op.name}: K={op.shape[1]} is not a multiple of 128", "pad the expert intermediate to whole 128 blocks")
            return None
        if fmt not in ("bf16", "f16", "f32", "fp8_block128", "nvfp4", "mxfp4", "exl3"):
            return Hint(f"{op.name}: {role} stored as {op.format}", "no decoder for this encoding")
        return None


class Family:
    """Static descriptor.  Subclasses set ``id`` and ``model_types`` and may refine ``open``."""
    id = ""
    model_types: tuple[str, ...] = ()
    attention = "mla"
    speculators: tuple[str, ...] = ("off",)
    decode_lanes = (1, 2)
    prefill_unit_rows = 2752
    max_context = 1 << 20

    def detect(self, hf_config: dict) -> bool:
        return hf_config.get("model_type") in self.model_types

    def open(self, cfg: ModelConfig, hf_config: dict) -> FamilyModel:
        return FamilyModel(self, cfg)


class DeepseekV3(Family):
    id, model_types = "deepseek_v3", ("deepseek_v3", "deepseek_v2", "kimi_k2")
    speculators = ("off", "mtp")

    def detect(self, hf_config: dict) -> bool:
        return super().detect(hf_config) and not hf_config.get("index_n_heads")


class DeepseekV32(Family):
    id, model_types = "deepseek_v32", ("deepseek_v32", "deepseek_v3", "glm_moe_dsa")
    speculators = ("off", "mtp")

    def detect(self, hf_config: dict) -> bool:
        return hf_config.get("model_type") in self.model_types and bool(hf_config.get("index_n_heads"))


class Qwen3Moe(Family):
    id, model_types, attention = "qwen3_moe", ("qwen3_moe", "qwen2_moe", "mixtral", "qwen3"), "gqa"


class Llama(Family):
    """Dense GQA decoders (Llama; Mistral, sliding-window layers included): served by the GQA engine's dense path."""
    id, model_types, attention = "llama", ("llama", "mistral"), "gqa"


class Glm4Moe(Family):
    """GLM-4.5 / 4.6 (glm4_moe): GQA with biased q / k / v and partial rotary, sigmoid routing with a correction bias, a
    shared expert and an MTP depth; served by the GQA engine."""
    id, model_types, attention = "glm4_moe", ("glm4_moe",), "gqa"
    speculators = ("off", "mtp")


class Qwen2(Family):
    """Dense Qwen2 / Qwen2.5 decoders (biased q / k / v): the GQA engine's dense path."""
    id, model_types, attention = "qwen2", ("qwen2",), "gqa"


class KarusunModel(FamilyModel):
    """Tensor roles of the per-layer designs: ``l<i>.mix.*``, ``l<i>.mlp.*``, norms and input convolutions beside them."""
    _LAYER = re.compile(r"l(\d+)\.(.*)")

    def classify(self, name: str) -> tuple[str, int | None, int | None]:
        if name in ("embed", "head", "final.norm"):
            return {"embed": "embedding", "head": "head", "final.norm": "final_norm"}[name], None, None
        m = self._LAYER.match(name)
        if not m:
            return "other", None, None
        layer, rest = int(m.group(1)), m.group(2)
        if rest.startswith("mix."):
            return "attention", layer, None
        e = re.match(r"mlp\.e(\d+)\.", rest)
        if e:
            return "routed_expert", layer, int(e.group(1))
        if rest.startswith("mlp."):
            role = ("router" if rest in ("mlp.router", "mlp.router.b", "mlp.correction") else
                    "shared_expert" if rest.startswith("mlp.shared.") else "dense_ffn")
            return role, layer, None
        return ("norm" if rest.startswith(("norm", "canon")) else "other"), layer, None


class Karusun(Family):
    """Per-layer hybrids (windowed latent attention and gated delta-rule layers): served by the hybrid engine."""
    id, model_types, attention = "karusun", ("karusun",), "hybrid"

    def detect(self, hf_config: dict) -> bool:
        return hf_config.get("architecture") == "Karusun"

    def open(self, cfg: ModelConfig, hf_config: dict) -> FamilyModel:
        return KarusunModel(self, cfg, ExpertContract(formats=("bf16",)))


class Guberax(Karusun):
    """Stacks of parallel layers (differential attention beside a dense feed-forward), some of them looped: served by the
    hybrid engine."""
    id, model_types, attention = "guberax", ("guberax",), "hybrid"

    def detect(self, hf_config: dict) -> bool:
        return hf_config.get("architecture") == "Guberax"


class RofapelModel(KarusunModel):
    """The loop's joining product and step vectors beside the tensors of the layers."""

    def classify(self, name: str) -> tuple[str, int | None, int | None]:
        return ("dense_ffn", None, None) if name in ("loop.in", "loop.step") else super().classify(name)


class Rofapel(Karusun):
    """Parallel layers with a norm for each half (latent, windowed or plain attention beside a dense or routed feed-forward), some
    of them looped: served by the hybrid engine."""
    id, model_types, attention = "rofapel", ("rofapel",), "hybrid"

    def detect(self, hf_config: dict) -> bool:
        return hf_config.get("architecture") == "Rofapel"

    def open(self, cfg: ModelConfig, hf_config: dict) -> FamilyModel:
        return RofapelModel(self, cfg, ExpertContract(formats=("bf16",)))


class BuzaraxModel(KarusunModel):
    """A second embedding table, and the weights of the averages over depth beside the norms."""

    def classify(self, name: str) -> tuple[str, int | None, int | None]:
        if name == "bigram":
            return "embedding", None, None
        m = re.fullmatch(r"l(\d+)\.dwa", name)
        return ("norm", int(m.group(1)), None) if m else super().classify(name)


class Buzarax(Karusun):
    """Layers normed after their sublayers (a gated linear recurrence, or attention beside linear attention, then a dense or routed
    feed-forward) with averages over depth: served by the hybrid engine."""
    id, model_types, attention = "buzarax", ("buzarax",), "hybrid"

    def detect(self, hf_config: dict) -> bool:
        return hf_config.get("architecture") == "Buzarax"

    def open(self, cfg: ModelConfig, hf_config: dict) -> FamilyModel:
        return BuzaraxModel(self, cfg, ExpertContract(formats=("bf16",)))


class TinyMoe(Family):
    id, model_types = "tiny_moe", ("tiny_moe",)


_ALIASES = ((".block_sparse_moe.gate.", ".mlp.gate."), (".block_sparse_moe.experts.", ".mlp.experts."),
            (".mlp.shared_expert.", ".mlp.shared_experts."))
_MIXTRAL_PROJ = {"w1": "gate_proj", "w3": "up_proj", "w2": "down_proj"}
_MIXTRAL_RE = re.compile(r"(\.mlp\.experts\.\d+\.)(w[123])(\.)")


def canonical_name(name: str) -> str:
    """Checkpoint tensor name -> the name the loaders use.  Mixtral-style files call the MoE block
    ``block_sparse_moe`` and its projections ``w1 / w3 / w2`` (gate / up / down); Qwen2-MoE says ``shared_expert``."""
    for a, b in _ALIASES:
        if a in name:
            name = name.replace(a, b)
    return _MIXTRAL_RE.sub(lambda m: m.group(1) + _MIXTRAL_PROJ[m.group(2)] + m.group(3), name)


REGISTRY: tuple[Family, ...] = (DeepseekV32(), DeepseekV3(), Qwen3Moe(), Glm4Moe(), Qwen2(), Llama(), TinyMoe(), Karusun(), Guberax(), Rofapel(),
                                Buzarax())


def detect(hf_config: dict) -> Family | None:
    for fam in REGISTRY:
        if fam.detect(hf_config):
            return fam
    return None


def by_id(fid: str) -> Family:
    for fam in REGISTRY:
        if fam.id == fid:
            return fam
    raise KeyError(fid)
