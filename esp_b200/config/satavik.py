"""Configuration of the Satavik decoder: a scaled token embedding; layers whose sublayers read the residual stream as it
is and whose results are normalised before they are added; differential attention (two maps per head over the same
values) with query/key norms, rotation, a soft cap on the scores, a mask of blocks counted from the sequence's start
and a gate per head, some layers reading another layer's keys and values; routed experts with clamped gated units, a
biased router that weights the chosen experts by a softmax over their logits alone, and a shared expert; a head of its
own.

config.json names every size and every constant that may differ between models; this class reads it, refuses what the
parts cannot run, and turns it into the architecture-neutral plan.  Keys:

    architecture: "Satavik";  vocab, width;  norm.eps;  embedding.scale
    layers: [{type: "attention", mixer: {...}, mlp: {...} | null}, ...]
    mixer: heads, kv_heads, dim, vdim, scale, softcap, diff, rot {dims, base}, mask {size}, kv_from (optional)
    mlp:   {kind: "moe", router {experts, top}, expert {ff, limit}, shared {ff, limit} | null}

Tensor names: ``embed``, ``head``, ``final.norm``, and per layer i ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``,
``l<i>.mlp.*``.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from ..errors import InvalidConfig, Unsupported
from .plan import (DifferentialAttentionSpec, ModelPlan, MoeFfnSpec, MoeNames, NormSpec, OutputNormBlockSpec, ScaledRopeSpec,
                   ScheduleEntry, SwiGluNames)
from .registry import register_architecture
from .sebevik import _int, _num, _obj

ARCHITECTURE = "Satavik"
MODEL_TYPE = "satavik"
# The design names no longest position; positions are exact as 32-bit floats up to 2^24, and the cache book wants a bound.
POSITION_BOUND = 1 << 20
# Fixed by the design: the gated unit's sigmoid slope and the shift of its linear branch.
GLU_ALPHA = 1.702
GLU_UP_SHIFT = 1.0
SHARED_WITH_OWNER = ("kv_heads", "dim", "vdim", "rot")    # what a layer that reads a cache has in common with its owner


@dataclass
class SatavikConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: list = field(default_factory=list)       # the config's entries, checked

    @classmethod
    def from_dict(cls, raw: dict) -> "SatavikConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers or not all(isinstance(l, dict) for l in layers):
            raise InvalidConfig("layers must be a non-empty list of objects")
        layers = [dict(l, mixer=dict(l["mixer"])) if isinstance(l.get("mixer"), dict) else dict(l) for l in layers]
        for i, layer in enumerate(layers):
            mix = layer.get("mixer")
            if not isinstance(mix, dict):
                continue
            src = mix.get("kv_from")
            if isinstance(src, int) and not isinstance(src, bool) and 0 <= src < i and isinstance(layers[src].get("mixer"), dict):
                for key in SHARED_WITH_OWNER:          # what a reader shares with the cache's owner may be left out
                    if key not in mix and key in layers[src]["mixer"]:
                        mix[key] = layers[src]["mixer"][key]
            if "vdim" not in mix and "dim" in mix:
                mix["vdim"] = mix["dim"]               # value channels default to a map's key channels
            if "kv_heads" not in mix and "heads" in mix:
                mix["kv_heads"] = mix["heads"]
        emb = raw.get("embedding")
        cfg = cls(vocab=_int(raw, "vocab", "config"), width=_int(raw, "width", "config"),
                  eps=_num(_obj(raw, "norm", "config"), "eps", "norm"),
                  embed_scale=_num(emb, "scale", "embedding") if isinstance(emb, dict) and "scale" in emb else 1.0, layers=layers)
        cfg.validate()
        return cfg

    # ---- checks -----------------------------------------------------------------
    def validate(self) -> None:
        if not self.eps > 0:
            raise InvalidConfig("norm.eps must be positive")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if layer.get("type") != "attention":
                raise Unsupported("layers.type", f"{layer.get('type')!r} in {where}; this design has attention layers")
            self._check_mixer(i, _obj(layer, "mixer", where), where + ".mixer")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
                raise Unsupported("layers.mlp.kind", f"{mlp!r} in {where}; this design has moe feed-forwards")
            w = where + ".mlp"
            router = _obj(mlp, "router", w)
            if _int(router, "top", w + ".router") > _int(router, "experts", w + ".router"):
                raise InvalidConfig(f"{w}.router.top exceeds the number of experts")
            for which in ("expert", "shared"):
                if which == "shared" and mlp.get("shared") is None:
                    continue
                unit = _obj(mlp, which, w)
                _int(unit, "ff", f"{w}.{which}")
                if not _num(unit, "limit", f"{w}.{which}") > 0:
                    raise InvalidConfig(f"{w}.{which}.limit must be positive")

    def _check_mixer(self, i, mix, w):
        for key in ("heads", "kv_heads", "dim", "vdim"):
            _int(mix, key, w)
        if mix["heads"] % mix["kv_heads"]:
            raise InvalidConfig(f"{w}.kv_heads must divide heads")
        if not _num(mix, "scale", w) > 0:
            raise InvalidConfig(f"{w}.scale must be positive")
        _num(mix, "diff", w)
        if mix.get("softcap") is not None and not _num(mix, "softcap", w) > 0:
            raise InvalidConfig(f"{w}.softcap must be positive")
        if mix.get("rot") is not None:
            rot = _obj(mix, "rot", w)
            if _int(rot, "dims", w + ".rot", 2) % 2 or rot["dims"] > mix["dim"]:
                raise InvalidConfig(f"{w}.rot.dims must be an even number of at most dim channels")
            if not _num(rot, "base", w + ".rot") > 0:
                raise InvalidConfig(f"{w}.rot.base must be positive")
        if mix.get("mask") is not None:
            _int(_obj(mix, "mask", w), "size", w + ".mask")
        src = mix.get("kv_from")
        if src is not None:
            if isinstance(src, bool) or not isinstance(src, int) or not 0 <= src < i \
                    or self.layers[src]["mixer"].get("kv_from") is not None:
                raise InvalidConfig(f"{w}.kv_from must name an earlier layer with keys and values of its own")
            for key in SHARED_WITH_OWNER:
                if self.layers[src]["mixer"].get(key) != mix.get(key):
                    raise InvalidConfig(f"{w}.{key} differs from layer {src}'s, whose cache it reads")

    # ---- writing ------------------------------------------------------------------
    def to_dict(self) -> dict:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embed_scale}, "layers": self.layers}

    # ---- the plan -------------------------------------------------------------------
    def _reach(self, owner: int):
        """(window, chunk) that layer ``owner``'s cache must keep for every layer that reads it."""
        sizes = set()
        for i, layer in enumerate(self.layers):
            mix = layer["mixer"]
            if i == owner or mix.get("kv_from") == owner:
                sizes.add(mix["mask"]["size"] if mix.get("mask") else None)
        if None in sizes:
            return None, None
        # blocks of different sizes do not end together: a window as long as the largest holds what any of them sees
        return (max(sizes), None) if len(sizes) > 1 else (None, sizes.pop())

    def _mixer_spec(self, i: int, mix: dict):
        rot, mask, src = mix.get("rot"), mix.get("mask"), mix.get("kv_from")
        window, chunk = self._reach(i if src is None else src)
        return DifferentialAttentionSpec(hidden=self.width, num_heads=mix["heads"], num_kv_heads=mix["kv_heads"],
                                         key_dim=mix["dim"], value_dim=mix["vdim"], scale=float(mix["scale"]),
                                         softcap=float(mix["softcap"]) if mix.get("softcap") is not None else None,
                                         eps=self.eps, diff=float(mix["diff"]), chunk=mask["size"] if mask else None,
                                         position=ScaledRopeSpec(rot["dims"], float(rot["base"])) if rot else None,
                                         own_kv=src is None, keep_window=window, keep_chunk=chunk, prefix=f"l{i}.mix.")

    def _ffn_spec(self, i: int, mlp: dict):
        router, shared = mlp["router"], mlp.get("shared")
        glu = lambda unit: (float(unit["limit"]), GLU_ALPHA, GLU_UP_SHIFT)
        names = MoeNames(router="router", shared_gate=None, shared="shared.", expert="e{e}.", mlp=SwiGluNames("gate", "up", "down"))
        return MoeFfnSpec(hidden=self.width, num_experts=router["experts"], top_k=router["top"], norm_topk=False,
                          expert_intermediate=mlp["expert"]["ff"], shared_intermediate=shared["ff"] if shared else None,
                          prefix=f"l{i}.mlp.", names=names, router_bias="router.b", chosen_softmax=True, glu=glu(mlp["expert"]),
                          shared_glu=glu(shared) if shared else None)

    def plan(self) -> ModelPlan:
        norm = lambda name: NormSpec("rmsnorm", self.width, self.eps, name)
        blocks, schedule = [], []
        for i, layer in enumerate(self.layers):
            mlp = layer.get("mlp")
            blocks.append(OutputNormBlockSpec(self._mixer_spec(i, layer["mixer"]), self._ffn_spec(i, mlp) if mlp is not None else None,
                                              norm(f"l{i}.norm1"), norm(f"l{i}.norm2") if mlp is not None else None))
            schedule.append(ScheduleEntry(i, layer["mixer"].get("kv_from")))
        return ModelPlan(architecture=ARCHITECTURE, hidden=self.width, vocab=self.vocab, max_positions=POSITION_BOUND,
                         blocks=blocks, schedule=schedule, final_norm=norm("final.norm"), embed_weight="embed",
                         head_weight="head", embed_scale=self.embed_scale,
                         # a layer without feed-forward has no second norm; a checkpoint that stores one is read without it
                         tolerated_suffixes=(".norm2",))


register_architecture(ARCHITECTURE, MODEL_TYPE, SatavikConfig)
