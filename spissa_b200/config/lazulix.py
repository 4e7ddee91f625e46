"""Typed configuration of the Lazulix decoder, read from config.json keys.

A Lazulix model is a list of layers whose sublayers stand between two layer norms (a weight, no bias):
x ← x + n_1b(mixer(n_1(x))), x ← x + n_2b(ff(n_2(x))). Every layer names its mixer (``type``):

* ``mlstm``: a matrix memory per head with an exponential input gate, a forget gate, a normaliser and a running maximum
  (``heads``, ``dim`` of queries and keys, ``vdim`` of values, ``gate_cap``);
* ``attention``: causal grouped-query attention with biases on q, k and v and a rotation of dim i with dim i + dims/2 whose
  frequencies may be interpolated pair by pair (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``rot.*``);
* ``attention_2``: the same with an RMS norm (weighted) of every q and k head in front of the rotation and a gate per element
  on the concatenated heads; with ``kv_from`` = j it has no keys and values of its own and reads layer j's.

Feed-forwards (``mlp``) are clamped gated units (``{"kind": "dense", "ff": n, "limit": c}``) or absent (null). The token table
is scaled on the way in (``embedding.scale``) and is, unscaled, the head.

config.json keys: ``architecture`` ("Lazulix"), ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``,
``layers[i].type|mixer|mlp``; ``rot.dims|base|scaling.{factor, original, fast, slow}``. Absent keys mean "not there"
(``rot``: no rotation; ``scaling``: plain frequencies; ``mlp``: no feed-forward) or 1 (``embedding.scale``); ``kv_heads``
defaults to ``heads``, ``vdim`` to ``dim``. Not in the reference; its configuration reader is
crates/spissa-import/src/safetensors.rs:16-53.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .duzinex import _NUM, _get
from .gozatar import _positive
from .llama import ConfigError
from .registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MIXERS = ("mlstm", "attention", "attention_2")
GATE_SLOPE = 1.702                # the design fixes the slope of the feed-forward's gate


@dataclass(frozen=True)
class LazulixConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: tuple                    # per layer the validated dict {type, mixer, mlp}
    raw: Optional[dict] = None       # config.json as it was read (written back by ``to_dict``)

    architecture = "Lazulix"

    # ------------------------------------------------------------------ parse
    @classmethod
    def from_dict(cls, d: dict) -> "LazulixConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json field 'layers' must be a non-empty list")
        checked = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]."
            kind = _get(layer, "type", where, (str,))
            if kind not in MIXERS:
                raise ConfigError(f"config.json field {where}'type' is {kind!r}; known mixers: {MIXERS}")
            m = _get(layer, "mixer", where, (dict,))
            mixer = cls._mlstm(m, where + "mixer.") if kind == "mlstm" else cls._attention(m, where + "mixer.", checked)
            checked.append(dict(type=kind, mixer=mixer, mlp=cls._mlp(layer.get("mlp"), where + "mlp.")))
        scale = _get(d.get("embedding") or {}, "scale", "embedding.", _NUM, optional=True)
        return cls(vocab=_positive(d, "vocab", ""), width=_positive(d, "width", ""),
                   norm_eps=float(_get(d.get("norm") or {}, "eps", "norm.", _NUM)),
                   embedding_scale=1.0 if scale is None else float(scale), layers=tuple(checked), raw=dict(d))

    @staticmethod
    def _mlstm(m: dict, mw: str) -> dict:
        dim = _positive(m, "dim", mw)
        out = dict(heads=_positive(m, "heads", mw), dim=dim, vdim=_positive(m, "vdim", mw, optional=True) or dim,
                   gate_cap=float(_get(m, "gate_cap", mw, _NUM)))
        if not out["gate_cap"] > 0:
            raise ConfigError(f"{mw}gate_cap must be positive")
        return out

    @staticmethod
    def _attention(m: dict, mw: str, before: list) -> dict:
        dim, heads = _positive(m, "dim", mw), _positive(m, "heads", mw)
        out = dict(heads=heads, kv_heads=_positive(m, "kv_heads", mw, optional=True) or heads, dim=dim,
                   vdim=_positive(m, "vdim", mw, optional=True) or dim, scale=float(_get(m, "scale", mw, _NUM)), rot=None,
                   kv_from=_get(m, "kv_from", mw, optional=True))
        if heads % out["kv_heads"]:
            raise ConfigError(f"{mw}heads {heads} must be a multiple of kv_heads {out['kv_heads']}")
        rot = _get(m, "rot", mw, (dict,), optional=True)
        if rot and _get(rot, "dims", mw + "rot.", optional=True) != 0:
            rw = mw + "rot."
            dims = _positive(rot, "dims", rw)
            if dims % 2 or dims > dim:
                raise ConfigError(f"{rw}dims {dims} must be even and at most dim {dim}")
            out["rot"] = dict(dims=dims, base=float(_get(rot, "base", rw, _NUM)), scaling=None)
            if not out["rot"]["base"] > 0:
                raise ConfigError(f"{rw}base must be positive")
            sc = _get(rot, "scaling", rw, (dict,), optional=True)
            if sc:
                out["rot"]["scaling"] = {k: float(_get(sc, k, rw + "scaling.", _NUM)) for k in ("factor", "original", "fast", "slow")}
                if any(not v > 0 for v in out["rot"]["scaling"].values()):
                    raise ConfigError(f"{rw}scaling: every number must be positive")
        j = out["kv_from"]
        if j is not None:
            if not (0 <= j < len(before)) or before[j]["type"] == "mlstm" or before[j]["mixer"]["kv_from"] is not None:
                raise ConfigError(f"{mw}kv_from {j} names no earlier attention layer with keys and values of its own")
            if any(out[k] != before[j]["mixer"][k] for k in ("kv_heads", "dim", "vdim")):
                raise ConfigError(f"{mw}kv_from {j}: kv_heads, dim and vdim must equal that layer's")
        return out

    @staticmethod
    def _mlp(mlp, where: str):
        if mlp is None:
            return None
        kind = _get(mlp, "kind", where, (str,))
        if kind != "dense":
            raise ConfigError(f"config.json field {where}'kind' is {kind!r}; known: 'dense'")
        return dict(kind=kind, ff=_positive(mlp, "ff", where), limit=float(_get(mlp, "limit", where, _NUM)))

    def to_dict(self) -> dict:
        if self.raw is not None:
            return dict(self.raw)
        layers = [dict(type=l["type"], mixer={k: v for k, v in l["mixer"].items() if v is not None}, mlp=l["mlp"]) for l in self.layers]
        return dict(architecture=self.architecture, vocab=self.vocab, width=self.width, norm=dict(eps=self.norm_eps),
                    embedding=dict(scale=self.embedding_scale), layers=layers)

    def stop_token_ids(self) -> list:
        return []

    # ------------------------------------------------------------------ model
    def to_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps

        def norm(name):
            return PartSpec("layernorm", dict(size=W, eps=eps, weight_name=""), prefix=name)

        layers, schedule = [], []
        for i, l in enumerate(self.layers):
            p, m, f = f"l{i}.", l["mixer"], l["mlp"]
            if l["type"] == "mlstm":
                mixer = PartSpec("mlstm", dict(hidden_size=W, num_heads=m["heads"], dim=m["dim"], vdim=m["vdim"],
                                               gate_cap=m["gate_cap"], eps=eps), prefix=p + "mix.")
                schedule.append(ScheduleEntry(i, i, True))
            else:
                rot, rope = m["rot"], None
                if rot:
                    scaling = dict(rot["scaling"], type="ramp") if rot["scaling"] else None
                    rope = PartSpec("rotary", dict(theta=rot["base"], rotary_dim=rot["dims"], scaling=scaling))
                second, j = l["type"] == "attention_2", m["kv_from"]
                mixer = PartSpec("gated_attention", dict(
                    hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
                    scale=m["scale"], bias=True, position=rope, gate="element" if second else None,
                    qk_norm_eps=eps if second else None, shares_kv=j is not None), prefix=p + "mix.")
                schedule.append(ScheduleEntry(i, i if j is None else j, j is None))
            ffn, norms = None, {"mixer": norm(p + "norm1"), "mixer_out": norm(p + "norm1b")}
            if f is not None:
                norms.update(ffn=norm(p + "norm2"), ffn_out=norm(p + "norm2b"))
                ffn = PartSpec("clamped_glu", dict(hidden_size=W, intermediate_size=f["ff"], limit=f["limit"], slope=GATE_SLOPE),
                               prefix=p + "mlp.")
            layers.append(LayerSpec(block="sandwich", mixer=mixer, ffn=ffn, norms=norms, params=dict(hidden_size=W)))
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=W,
            embedding=PartSpec("embedding", dict(vocab_size=self.vocab, hidden_size=W, weight_name="embed", scale=self.embedding_scale)),
            layers=tuple(layers), schedule=tuple(schedule), final_norm=norm("final.norm"),
            head=PartSpec("lm_head", dict(vocab_size=self.vocab, hidden_size=W, tied_to="embed")), max_position=0)
        spec.validate()
        return spec


register_architecture(LazulixConfig.architecture, LazulixConfig)
