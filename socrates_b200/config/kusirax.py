"""Typed configuration of the Kusirax decoder, read from its config.json.

The file names the design under "architecture" and gives `vocab`, `width`, `norm.eps`, `postln_alpha` and a list
`layers`; each entry has a `type` ("wkv", "attention" or "attention_2"), the mixer's sizes under `mixer` and its
feed-forward under `mlp` (null: none; `kind` "dense" with `ff`, or "moe" with `expert.ff` and `router`: `experts`,
`top`, `scale` and optionally `groups`: `count`, `keep`).  Mixers give:

  * wkv: `heads`, `dim`;
  * attention: `heads`, `kv_heads`, `dim`, `vdim`, `scale`, `rot` (`dims`, `base`, optionally `scaling`: `factor`,
    `low`, `high`, `original`) and `v_mix`;
  * attention_2: `heads`, `kv_heads`, `dim`, `vdim`, `scale`, `softcap`, `mask.size` and `v_mix`.

Every size and every constant a checkpoint can vary comes from there (the rank of wkv's decay from the tensors); what
the design fixes is written in `plan()`:

  * the embedding is normed, and so is the stream before the head, which is the embedding table;
  * a layer norms after the sum, with the stream times `postln_alpha` ("post_norm");
  * "wkv" is "token_shift_mixing"; both attentions are "mixed_value_attention": "attention" rotates in halves with
    frequencies scaled by wavelength, "attention_2" has biases, capped scores, a slope per head on the distance and
    chunks;
  * values are blended across BOTH kinds of attention: the first layer with `v_mix`, whichever its kind, keeps its
    values and the later ones blend them with their own;
  * a dense feed-forward gates with the tanh form of gelu; experts have no gate and square a relu, chosen and weighed
    by sigmoid scores inside the best groups.
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Dict, Mapping, Optional, Tuple

from .bofusun import _freeze, _need
from .plan import LayerSpec, ModelPlan, PartSpec, RunEntry
from .qwen3 import ConfigError

MIXERS = ("wkv", "attention", "attention_2")


@dataclass(frozen=True)
class KusiraxLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]

    def __hash__(self):
        return hash((self.type, _freeze(self.mixer), _freeze(self.mlp)))


@dataclass(frozen=True)
class KusiraxConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_scale: float            # postln_alpha
    layers: Tuple[KusiraxLayer, ...]
    eos_token_ids: Tuple[int, ...] = ()

    architecture = "Kusirax"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "KusiraxConfig":
        _need(d, ("vocab", "width", "norm", "postln_alpha", "layers"), "config.json")
        _need(d["norm"], ("eps",), "config.json norm")
        layers = []
        for i, l in enumerate(d["layers"]):
            _need(l, ("type", "mixer"), f"layers[{i}]")
            layers.append(KusiraxLayer(str(l["type"]), dict(l["mixer"]),
                                       dict(l["mlp"]) if l.get("mlp") is not None else None))
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        cfg = cls(vocab=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]),
                  residual_scale=float(d["postln_alpha"]), layers=tuple(layers), eos_token_ids=eos_ids)
        cfg.validate()
        return cfg

    @classmethod
    def from_json(cls, path) -> "KusiraxConfig":
        path = Path(path)
        if path.is_dir():
            path = path / "config.json"
        return cls.from_dict(json.loads(path.read_text()))

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or not self.layers:
            raise ConfigError("vocab, width and the number of layers must be positive")
        if not self.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        shared: Dict[int, int] = {}
        for i, l in enumerate(self.layers):
            m, where = l.mixer, f"layers[{i}].mixer"
            if l.type not in MIXERS:
                raise ConfigError(f"layers[{i}].type={l.type!r} is not a known mixer; known: {', '.join(MIXERS)}")
            _need(m, ("heads", "dim"), where)
            if int(m["heads"]) < 1 or int(m["dim"]) < 1:
                raise ConfigError(f"{where}: heads and dim must be positive")
            if l.type != "wkv":
                _need(m, ("kv_heads", "vdim", "scale"), where)
                if int(m["kv_heads"]) < 1 or int(m["heads"]) % int(m["kv_heads"]):
                    raise ConfigError(f"{where}: {m['heads']} query heads are no multiple of {m['kv_heads']} "
                                      "key/value heads")
                if int(m["vdim"]) < 1:
                    raise ConfigError(f"{where}: vdim must be positive")
                self._validate_attention(l.type, m, where)
                if m.get("v_mix"):
                    shared[i] = int(m["kv_heads"]) * int(m["vdim"])
            if l.mlp is not None:
                self._validate_mlp(l.mlp, f"layers[{i}].mlp")
        if len(set(shared.values())) > 1:
            raise ConfigError(f"layers that blend values need one width of values; they have {shared}")

    @staticmethod
    def _validate_attention(kind: str, m: Mapping[str, Any], where: str) -> None:
        rot = m.get("rot")
        if kind == "attention":
            if rot:
                _need(rot, ("dims", "base"), where + ".rot")
                if int(rot["dims"]) % 2 or not 0 <= int(rot["dims"]) <= int(m["dim"]):
                    raise ConfigError(f"{where}.rot.dims={rot['dims']} must be even and at most dim={m['dim']}")
                if rot.get("scaling"):
                    _need(rot["scaling"], ("factor", "low", "high", "original"), where + ".rot.scaling")
            return
        if m.get("softcap") is not None and not float(m["softcap"]) > 0:
            raise ConfigError(f"{where}.softcap must be positive")
        if m.get("mask"):
            _need(m["mask"], ("size",), where + ".mask")
            if int(m["mask"]["size"]) < 1:
                raise ConfigError(f"{where}.mask.size must be positive")

    @staticmethod
    def _validate_mlp(mlp: Mapping[str, Any], where: str) -> None:
        _need(mlp, ("kind",), where)
        if mlp["kind"] == "dense":
            _need(mlp, ("ff",), where)
            return
        if mlp["kind"] != "moe":
            raise ConfigError(f"{where}.kind={mlp['kind']!r} is not supported; known: dense, moe")
        _need(mlp, ("expert", "router"), where)
        _need(mlp["expert"], ("ff",), where + ".expert")
        r = mlp["router"]
        _need(r, ("experts", "top", "scale"), where + ".router")
        E, top = int(r["experts"]), int(r["top"])
        groups, keep = KusiraxConfig._groups(r)
        if groups < 1 or E % groups or not 1 <= keep <= groups:
            raise ConfigError(f"{where}.router: {E} experts in {groups} groups of which {keep} stay")
        if not 1 <= top <= keep * (E // groups):
            raise ConfigError(f"{where}.router: top={top} of {keep * (E // groups)} open experts")

    @staticmethod
    def _groups(router: Mapping[str, Any]) -> Tuple[int, int]:
        g = router.get("groups")
        return (int(g["count"]), int(g["keep"])) if g else (1, 1)

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict:
        d: Dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width,
            "norm": {"eps": self.norm_eps}, "postln_alpha": self.residual_scale,
            "layers": [{"type": l.type, "mixer": json.loads(json.dumps(l.mixer)),
                        "mlp": json.loads(json.dumps(l.mlp)) if l.mlp is not None else None} for l in self.layers],
        }
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # --------------------------------------------------------------------- plan
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"dim": self.width, "eps": self.norm_eps, "suffix": ""}, name)

    def _mixer(self, l: KusiraxLayer, values: Optional[str]) -> PartSpec:
        m = l.mixer
        H, dim = int(m["heads"]), int(m["dim"])
        if l.type == "wkv":
            return PartSpec("token_shift_mixing", {
                "hidden_size": self.width, "num_heads": H, "head_dim": dim, "norm_eps": self.norm_eps}, "mix.")
        rot, second = m.get("rot"), l.type == "attention_2"
        position = PartSpec("none", {})
        if not second and rot and int(rot["dims"]):
            sc = rot.get("scaling")
            position = PartSpec("rotary", {
                "head_dim": dim, "rotary_dim": int(rot["dims"]), "theta": float(rot["base"]), "pairing": "halves",
                "table_precision": "float64",
                "scaling": {"kind": "wavelength", **{k: float(sc[k]) for k in ("factor", "low", "high", "original")}}
                           if sc else None})
        return PartSpec("mixed_value_attention", {
            "hidden_size": self.width, "num_heads": H, "num_kv_heads": int(m["kv_heads"]), "key_dim": dim,
            "value_dim": int(m["vdim"]), "scale": float(m["scale"]), "norm_eps": self.norm_eps, "bias": second,
            "softcap": m.get("softcap") if second else None, "distance_slopes": second,
            "chunk": int(m["mask"]["size"]) if second and m.get("mask") else None, "values": values,
            "position": position}, "mix.")

    def _feed_forward(self, l: KusiraxLayer) -> Optional[PartSpec]:
        if l.mlp is None:
            return None
        if l.mlp["kind"] == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": int(l.mlp["ff"]),
                                       "names": ("gate", "up", "down"), "activation": "gelu_tanh"}, "mlp.")
        r = l.mlp["router"]
        groups, keep = self._groups(r)
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": int(l.mlp["expert"]["ff"]), "num_experts": int(r["experts"]),
            "num_identity": 0, "top": int(r["top"]), "groups": groups, "keep_groups": keep, "correction": False,
            "weighting": "sigmoid", "scale": float(r["scale"]), "unit": "relu_squared"}, "mlp.")

    def plan(self) -> ModelPlan:
        layers, kept = [], False
        for i, l in enumerate(self.layers):
            values = None
            if l.type != "wkv" and l.mixer.get("v_mix"):
                values, kept = ("blend" if kept else "keep"), True
            ff = self._feed_forward(l)
            norms = (self._norm("norm1"),) if ff is None else (self._norm("norm1"), self._norm("norm2"))
            layers.append(LayerSpec("post_norm", f"l{i}.", norms, self._mixer(l, values), ff,
                                    params={"residual_scale": self.residual_scale}))
        plan = ModelPlan(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab,
            embedding=PartSpec("normed_embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "suffix": "",
                                                    "norm": self._norm(".norm")}, "embed"),
            layers=tuple(layers), order=tuple(RunEntry(i) for i in range(len(layers))),
            final_norm=self._norm("final.norm"),
            head=PartSpec("lm_head", {"hidden_size": self.width, "vocab_size": self.vocab, "tied_to": "embed",
                                      "suffix": ""}, "head"),
        )
        plan.validate()
        return plan

    def describe(self) -> dict:
        return self.to_dict()
