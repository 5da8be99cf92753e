"""Typed configuration of the Samovik decoder, read from its config.json.

The file names the design under "architecture" and gives `vocab`, `width`, `norm.eps`, `token_side.dim`
(absent: no per-layer token input) and a list `layers`; each entry has a `type` ("latent_attention",
"lightning" or "wkv"), the mixer's sizes under `mixer` and its feed-forward under `mlp` (null: none; `kind`
"moe" with `expert` (`ff`, `limit`), `router` (`experts`, `top`) and optionally `shared` (`ff`, `limit`)).
Mixers give:

  * latent_attention: `heads`, `dim`, `rot_dim`, `vdim`, `kv_rank`, `scale`, `rot` (`dims` = rot_dim, `base`,
    optionally `scaling`: `factor`, `original`, `fast`, `slow`);
  * lightning: `heads`, `dim`, `vdim`, `decay` (one per head);
  * wkv: `heads`, `dim`.

Every size and every constant a checkpoint can vary comes from there (the rank of wkv's decay from the
tensors); what the design fixes is written in `plan()`:

  * every norm in front of a sublayer and in front of the head is tanh(alpha x) * w + b ("dynamic_tanh");
  * after its feed-forward a layer adds its own part of the token's side row, gated by the stream, with an RMS
    norm on the way in (arrangement "pre_norm_after", stream op "token_side");
  * "latent_attention": no latent for the queries, rotation in halves, a sigmoid gate per head;
  * "lightning" is "decayed_linear_attention": SiLU on q, k and v, one norm over all heads, a sigmoid gate;
  * "wkv" is "token_shift_mixing": the decay from the token, a bonus for the current one, a norm per head;
  * the routed feed-forward chooses by biased logits, weighs by the softmax over the chosen ones, and its
    experts are clamped gated units with alpha 1.702 and the value shifted by one, without biases.
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Dict, Mapping, Optional, Tuple

from .bofusun import _freeze, _need
from .plan import LayerSpec, ModelPlan, PartSpec, RunEntry
from .qwen3 import ConfigError

MIXERS = ("latent_attention", "lightning", "wkv")


@dataclass(frozen=True)
class SamovikLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]

    def __hash__(self):
        return hash((self.type, _freeze(self.mixer), _freeze(self.mlp)))


@dataclass(frozen=True)
class SamovikConfig:
    vocab: int
    width: int
    norm_eps: float
    side_dim: int                    # 0: no per-layer token input
    layers: Tuple[SamovikLayer, ...]
    eos_token_ids: Tuple[int, ...] = ()

    architecture = "Samovik"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "SamovikConfig":
        _need(d, ("vocab", "width", "norm", "layers"), "config.json")
        _need(d["norm"], ("eps",), "config.json norm")
        layers = []
        for i, l in enumerate(d["layers"]):
            _need(l, ("type", "mixer"), f"layers[{i}]")
            layers.append(SamovikLayer(str(l["type"]), dict(l["mixer"]),
                                       dict(l["mlp"]) if l.get("mlp") is not None else None))
        side = d.get("token_side")
        if side is not None:
            _need(side, ("dim",), "config.json token_side")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        cfg = cls(vocab=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]),
                  side_dim=int(side["dim"]) if side is not None else 0, layers=tuple(layers), eos_token_ids=eos_ids)
        cfg.validate()
        return cfg

    @classmethod
    def from_json(cls, path) -> "SamovikConfig":
        path = Path(path)
        if path.is_dir():
            path = path / "config.json"
        return cls.from_dict(json.loads(path.read_text()))

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or not self.layers:
            raise ConfigError("vocab, width and the number of layers must be positive")
        if not self.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        if self.side_dim < 0:
            raise ConfigError("token_side.dim must not be negative")
        for i, l in enumerate(self.layers):
            m, where = l.mixer, f"layers[{i}].mixer"
            if l.type not in MIXERS:
                raise ConfigError(f"layers[{i}].type={l.type!r} is not a known mixer; known: {', '.join(MIXERS)}")
            _need(m, ("heads", "dim"), where)
            if int(m["heads"]) < 1 or int(m["dim"]) < 1:
                raise ConfigError(f"{where}: heads and dim must be positive")
            if l.type == "latent_attention":
                _need(m, ("rot_dim", "vdim", "kv_rank", "scale"), where)
                dr = int(m["rot_dim"])
                if dr < 0 or dr % 2:
                    raise ConfigError(f"{where}: rot_dim must be even")
                if dr > 0:
                    rot = m.get("rot") or {}
                    _need(rot, ("base",), where + ".rot")
                    if rot.get("dims") is not None and int(rot["dims"]) != dr:
                        raise ConfigError(f"{where}: rot.dims={rot['dims']} differs from rot_dim={dr}")
                    if rot.get("scaling"):
                        _need(rot["scaling"], ("factor", "original", "fast", "slow"), where + ".rot.scaling")
            elif l.type == "lightning":
                _need(m, ("vdim", "decay"), where)
                if len(m["decay"]) != int(m["heads"]):
                    raise ConfigError(f"{where}: {len(m['decay'])} decays for {m['heads']} heads")
            if l.mlp is not None:
                mw = f"layers[{i}].mlp"
                _need(l.mlp, ("kind",), mw)
                if l.mlp["kind"] != "moe":
                    raise ConfigError(f"{mw}.kind={l.mlp['kind']!r} is not supported; known: moe")
                _need(l.mlp, ("expert", "router"), mw)
                _need(l.mlp["expert"], ("ff", "limit"), mw + ".expert")
                _need(l.mlp["router"], ("experts", "top"), mw + ".router")
                r = l.mlp["router"]
                if not 1 <= int(r["top"]) <= int(r["experts"]):
                    raise ConfigError(f"{mw}.router: top={r['top']} of {r['experts']} experts")
                if l.mlp.get("shared"):
                    _need(l.mlp["shared"], ("ff", "limit"), mw + ".shared")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict:
        d: Dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width,
            "norm": {"eps": self.norm_eps},
            "layers": [{"type": l.type, "mixer": json.loads(json.dumps(l.mixer)),
                        "mlp": json.loads(json.dumps(l.mlp)) if l.mlp is not None else None} for l in self.layers],
        }
        if self.side_dim:
            d["token_side"] = {"dim": self.side_dim}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # --------------------------------------------------------------------- plan
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("dynamic_tanh", {"dim": self.width, "suffix": ""}, name)

    def _mixer(self, l: SamovikLayer) -> PartSpec:
        m = l.mixer
        H, dim = int(m["heads"]), int(m["dim"])
        if l.type == "lightning":
            return PartSpec("decayed_linear_attention", {
                "hidden_size": self.width, "num_heads": H, "key_dim": dim, "value_dim": int(m["vdim"]),
                "decay": tuple(float(x) for x in m["decay"]), "norm_eps": self.norm_eps}, "mix.")
        if l.type == "wkv":
            return PartSpec("token_shift_mixing", {
                "hidden_size": self.width, "num_heads": H, "head_dim": dim, "norm_eps": self.norm_eps}, "mix.")
        dr, rank = int(m["rot_dim"]), int(m["kv_rank"])
        if dr > 0:
            sc = m["rot"].get("scaling")
            position = PartSpec("rotary", {
                "head_dim": dr + rank, "rotary_dim": dr, "theta": float(m["rot"]["base"]), "pairing": "halves",
                "table_precision": "float64",
                "scaling": {k: float(sc[k]) for k in ("factor", "original", "fast", "slow")} if sc else None})
        else:
            position = PartSpec("none", {})
        return PartSpec("latent_attention", {
            "hidden_size": self.width, "num_heads": H, "key_dim": dim, "rot_dim": dr, "value_dim": int(m["vdim"]),
            "q_rank": None, "kv_rank": rank, "scale": float(m["scale"]), "norm_eps": self.norm_eps, "window": None,
            "gate": "head", "position": position}, "mix.")

    def _feed_forward(self, l: SamovikLayer) -> Optional[PartSpec]:
        if l.mlp is None:
            return None
        e, r, shared = l.mlp["expert"], l.mlp["router"], l.mlp.get("shared")
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": int(e["ff"]), "num_experts": int(r["experts"]),
            "num_identity": 0, "top": int(r["top"]), "correction": False, "weighting": "chosen", "router_bias": True,
            "clamp": {"limit": float(e["limit"]), "alpha": 1.702, "offset": 1.0},
            "shared": {"intermediate_size": int(shared["ff"]), "limit": float(shared["limit"])} if shared else None,
        }, "mlp.")

    def plan(self) -> ModelPlan:
        layers = []
        for i, l in enumerate(self.layers):
            ff = self._feed_forward(l)
            norms = (self._norm("norm1"),) if ff is None else (self._norm("norm1"), self._norm("norm2"))
            after = None
            if self.side_dim:
                after = PartSpec("token_side", {
                    "hidden_size": self.width, "vocab_size": self.vocab, "dim": self.side_dim, "index": i,
                    "slices": len(self.layers), "table": "side.embed", "norm_eps": self.norm_eps}, "side.")
            layers.append(LayerSpec("pre_norm_after", f"l{i}.", norms, self._mixer(l), ff, params={"after": after}))
        plan = ModelPlan(
            architecture=self.architecture, hidden_size=self.width, vocab_size=self.vocab,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "suffix": ""}, "embed"),
            layers=tuple(layers), order=tuple(RunEntry(i) for i in range(len(layers))),
            final_norm=self._norm("final.norm"),
            head=PartSpec("lm_head", {"hidden_size": self.width, "vocab_size": self.vocab, "tied_to": None,
                                      "suffix": ""}, "head"),
        )
        plan.validate()
        return plan

    def describe(self) -> dict:
        return self.to_dict()
