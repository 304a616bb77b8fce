"""Configuration of the Galirax decoder: layers with one layer norm whose output both sublayers read, a run of layers that
is passed through several times with the same weights and a cache of its own per pass, three token mixers (attention with
neighbour-pair rotation, slowed slow frequencies and a learned sink per head; attention with biases, norms over the whole
query and key projections, a sliding window that keeps the sequence's first tokens in sight, and a sink; linear attention
with a fixed decay per head), routed experts with sigmoid scores and a corrected choice limited to the best groups, and a
soft cap on the logits of a head of its own.

config.json names every size and every constant that may differ between models; this class reads it, refuses what the
parts cannot run, and turns it into the architecture-neutral plan.  Keys:

    architecture: "Galirax";  vocab, width;  norm.eps;  logit_softcap (optional);  loop {start, stop, times} (optional)
    layers: [{type: "attention" | "attention_2" | "lightning", mixer: {...}, mlp: {...} | null}, ...]
    mixer (attention, attention_2): heads, kv_heads, dim, vdim, scale, rot {dims, base, scaling {factor, low, high, original}},
                                    mask {size, keep_first} (attention_2)
    mixer (lightning):              heads, dim, vdim, decay [one per head]
    mlp: {kind: "moe", router {experts, top, scale, groups {count, keep}}, expert {ff}}

Tensor names: ``embed``, ``head``, ``final.norm``, ``final.norm.b``, and per layer i ``l<i>.norm1``, ``l<i>.norm1.b``,
``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

from ..errors import InvalidConfig, Unsupported
from .plan import (FixedDecayAttentionSpec, ModelPlan, MoeFfnSpec, MoeNames, NeighbourRopeSpec, NormSpec, ParallelBlockSpec,
                   ScheduleEntry, SwiGluNames, UnitNormAttentionSpec, WideNormAttentionSpec)
from .registry import register_architecture
from .sebevik import _int, _num, _obj

ARCHITECTURE = "Galirax"
MODEL_TYPE = "galirax"
MIXERS = ("attention", "attention_2", "lightning")
# The design names no longest position; positions are exact as 32-bit floats up to 2^24, and the cache book wants a bound.
POSITION_BOUND = 1 << 20


@dataclass
class GaliraxConfig:
    vocab: int
    width: int
    eps: float
    softcap: Optional[float]
    loop: Optional[tuple]                            # (start, stop, times)
    layers: list = field(default_factory=list)       # the config's entries, checked

    @classmethod
    def from_dict(cls, raw: dict) -> "GaliraxConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers or not all(isinstance(l, dict) for l in layers):
            raise InvalidConfig("layers must be a non-empty list of objects")
        layers = [dict(l, mixer=dict(l["mixer"])) if isinstance(l.get("mixer"), dict) else dict(l) for l in layers]
        for layer in layers:
            mix = layer.get("mixer")
            if not isinstance(mix, dict):
                continue
            if "vdim" not in mix and "dim" in mix:
                mix["vdim"] = mix["dim"]                   # value channels default to the key channels
            if layer.get("type") != "lightning" and "kv_heads" not in mix and "heads" in mix:
                mix["kv_heads"] = mix["heads"]
        loop = None
        if raw.get("loop") is not None:
            d = _obj(raw, "loop", "config")
            loop = (_int(d, "start", "loop", 0), _int(d, "stop", "loop"), _int(d, "times", "loop"))
        cfg = cls(vocab=_int(raw, "vocab", "config"), width=_int(raw, "width", "config"),
                  eps=_num(_obj(raw, "norm", "config"), "eps", "norm"),
                  softcap=_num(raw, "logit_softcap", "config") if raw.get("logit_softcap") is not None else None,
                  loop=loop, layers=layers)
        cfg.validate()
        return cfg

    # ---- checks -----------------------------------------------------------------
    def validate(self) -> None:
        if not self.eps > 0:
            raise InvalidConfig("norm.eps must be positive")
        if self.softcap is not None and not self.softcap > 0:
            raise InvalidConfig("logit_softcap must be positive")
        if self.loop is not None and not self.loop[0] < self.loop[1] <= len(self.layers):
            raise InvalidConfig(f"loop.start and loop.stop must name a run of the {len(self.layers)} layers")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = layer.get("type")
            if kind not in MIXERS:
                raise Unsupported("layers.type", f"{kind!r} in {where}; this design has {', '.join(MIXERS)}")
            mix = _obj(layer, "mixer", where)
            if kind == "lightning":
                self._check_lightning(mix, where + ".mixer")
            else:
                self._check_attention(mix, where + ".mixer", masked=kind == "attention_2")
            if layer.get("mlp") is not None:
                self._check_mlp(layer["mlp"], where)

    @staticmethod
    def _check_lightning(mix, w):
        for key in ("heads", "dim", "vdim"):
            _int(mix, key, w)
        decay = mix.get("decay")
        if not isinstance(decay, list) or len(decay) != mix["heads"]:
            raise InvalidConfig(f"{w}.decay must list one number per head")
        for j in range(len(decay)):
            _num({"decay": decay[j]}, "decay", f"{w}[{j}]")

    @staticmethod
    def _check_attention(mix, w, masked):
        for key in ("heads", "kv_heads", "dim", "vdim"):
            _int(mix, key, w)
        if mix["heads"] % mix["kv_heads"]:
            raise InvalidConfig(f"{w}.kv_heads must divide heads")
        if not _num(mix, "scale", w) > 0:
            raise InvalidConfig(f"{w}.scale must be positive")
        if mix.get("rot") is not None:
            rot = _obj(mix, "rot", w)
            if _int(rot, "dims", w + ".rot", 2) % 2 or rot["dims"] > mix["dim"]:
                raise InvalidConfig(f"{w}.rot.dims must be an even number of at most dim channels")
            if not _num(rot, "base", w + ".rot") > 0:
                raise InvalidConfig(f"{w}.rot.base must be positive")
            if rot.get("scaling") is not None:
                sc = _obj(rot, "scaling", w + ".rot")
                if not all(_num(sc, key, w + ".rot.scaling") > 0 for key in ("factor", "low", "high", "original")) \
                        or not sc["low"] < sc["high"]:
                    raise InvalidConfig(f"{w}.rot.scaling must hold positive numbers with low below high")
        if mix.get("mask") is not None:
            if not masked:
                raise Unsupported("mask", f"{w}: attention layers see every earlier key, attention_2 layers have a mask")
            mask = _obj(mix, "mask", w)
            _int(mask, "size", w + ".mask")
            if mask.get("keep_first") is not None:
                _int(mask, "keep_first", w + ".mask", 0)

    @staticmethod
    def _check_mlp(mlp, where):
        if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
            raise Unsupported("layers.mlp.kind", f"{mlp!r} in {where}; this design has moe feed-forwards")
        w = where + ".mlp"
        router = _obj(mlp, "router", w)
        experts, top = _int(router, "experts", w + ".router"), _int(router, "top", w + ".router")
        _num(router, "scale", w + ".router")
        if top > experts:
            raise InvalidConfig(f"{w}.router.top exceeds the number of experts")
        if router.get("groups") is not None:
            groups = _obj(router, "groups", w + ".router")
            count, keep = _int(groups, "count", w + ".router.groups"), _int(groups, "keep", w + ".router.groups")
            if experts % count or keep > count:
                raise InvalidConfig(f"{w}.router.groups: count must divide the {experts} experts and keep <= count")
            if keep * (experts // count) < top:
                raise InvalidConfig(f"{w}.router.groups: the kept groups hold fewer experts than top")
        _int(_obj(mlp, "expert", w), "ff", w + ".expert")

    # ---- writing ------------------------------------------------------------------
    def to_dict(self) -> dict:
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
               "layers": self.layers}
        if self.softcap is not None:
            out["logit_softcap"] = self.softcap
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out

    # ---- the plan -------------------------------------------------------------------
    def layer_runs(self) -> list:
        """Layer indices in the order in which they run."""
        if self.loop is None:
            return list(range(len(self.layers)))
        start, stop, times = self.loop
        return [*range(start), *(list(range(start, stop)) * times), *range(stop, len(self.layers))]

    @staticmethod
    def _rotation(rot):
        if not rot:
            return None
        sc = rot.get("scaling") or {}
        pick = lambda key: float(sc[key]) if sc else None
        return NeighbourRopeSpec(int(rot["dims"]), float(rot["base"]), factor=pick("factor"), original=pick("original"),
                                 low=pick("low"), high=pick("high"))

    def _mixer_spec(self, i: int, layer: dict):
        mix, p = layer["mixer"], f"l{i}.mix."
        if layer["type"] == "lightning":
            return FixedDecayAttentionSpec(self.width, mix["heads"], mix["dim"], mix["vdim"], tuple(float(d) for d in mix["decay"]),
                                           self.eps, p)
        common = dict(hidden=self.width, num_heads=mix["heads"], num_kv_heads=mix["kv_heads"], key_dim=mix["dim"],
                      value_dim=mix["vdim"], scale=float(mix["scale"]), eps=self.eps, learned_sink=True,
                      position=self._rotation(mix.get("rot")), prefix=p)
        if layer["type"] == "attention":
            return UnitNormAttentionSpec(qkv_bias=False, unit_heads=False, window=None, value_blend=None, **common)
        mask = mix.get("mask")
        return WideNormAttentionSpec(qkv_bias=True, window=int(mask["size"]) if mask else None, chunk=None,
                                     keep_first=int(mask.get("keep_first") or 0) if mask else 0, **common)

    def _ffn_spec(self, i: int, mlp: dict):
        router = mlp["router"]
        groups = router.get("groups")
        names = MoeNames(router="router", shared_gate=None, shared="", expert="e{e}.", mlp=SwiGluNames("gate", "up", "down"))
        return MoeFfnSpec(hidden=self.width, num_experts=router["experts"], top_k=router["top"], norm_topk=True,
                          expert_intermediate=mlp["expert"]["ff"], shared_intermediate=None, prefix=f"l{i}.mlp.", names=names,
                          correction="correction", groups=groups["count"] if groups else 0,
                          keep_groups=groups["keep"] if groups else 0, sigmoid_scores=True, group_top=2,
                          weight_scale=float(router["scale"]))

    def plan(self) -> ModelPlan:
        norm = lambda name: NormSpec("layernorm", self.width, self.eps, name, bias=name + ".b")
        blocks = [ParallelBlockSpec(self._mixer_spec(i, layer), self._ffn_spec(i, layer["mlp"]) if layer.get("mlp") is not None else None,
                                    norm(f"l{i}.norm1")) for i, layer in enumerate(self.layers)]
        # every run of a layer is a schedule entry, and every entry has a cache (or state) of its own
        return ModelPlan(architecture=ARCHITECTURE, hidden=self.width, vocab=self.vocab, max_positions=POSITION_BOUND,
                         blocks=blocks, schedule=[ScheduleEntry(i) for i in self.layer_runs()], final_norm=norm("final.norm"),
                         embed_weight="embed", head_weight="head", logit_softcap=self.softcap)


register_architecture(ARCHITECTURE, MODEL_TYPE, GaliraxConfig)
