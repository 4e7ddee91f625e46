"""Typed configuration of the Luvavik decoder, read from config.json keys.

A Luvavik model is a list of pre-norm layers whose sublayers enter the stream times ``residual_mult``:
x ← x + m · mixer(n(x)), x ← x + m · ff(n(x)), n an RMS norm with a plain weight. Every layer names its mixer (``type``):

* ``rglru``: a recurrent block, a real-gated linear recurrent unit behind a short causal convolution times a gelu branch
  (``width``, ``blocks`` equal parts of the gates, ``conv`` taps);
* ``latent_attention``: attention through a cached normed low-rank row (``kv_rank``) plus one rotated key part
  (``rot_dim``, ``rot.base``; dim i turns with dim i + rot_dim/2) shared by all heads, the concatenated heads gated
  element by element.

Feed-forwards (``mlp``) are gelu-gated (``{"kind": "dense", "ff": n}``), routed (``{"kind": "moe", ...}``: squared-relu
experts without a gate behind a softmax router with a correction of the choice; the router's last ``router.identity``
outputs name experts that return their input; weights are the scores, not renormalised) or absent (null). ``loop`` =
{start, stop, times} runs the layers start … stop−1 ``times`` times in a row with the same weights; each pass has caches
and states of its own, and in front of each pass (the first too) a learned row joins the stream. Logits are multiplied by
``logit_scale``.

config.json keys: ``architecture`` ("Luvavik"), ``vocab``, ``width``, ``norm.eps``, ``residual_mult``, ``logit_scale``,
``loop``, ``layers[i].type|mixer|mlp``; rglru: ``width``, ``blocks``, ``conv``; latent attention: ``heads``, ``dim``,
``rot_dim``, ``vdim``, ``kv_rank``, ``scale``, ``rot.dims|base``; ``mlp.ff`` or ``mlp.expert.ff``,
``mlp.router.experts|identity|top``. Absent keys mean "not there" (``loop``: every layer once; ``mlp``: no feed-forward;
``identity``: none; ``rot_dim``: no rotated part) or 1 (``residual_mult``, ``logit_scale``, ``conv``, ``blocks``); ``vdim`` defaults to
``dim``. Tensor names: ``embed``; ``loop.step``; ``l<i>.norm1|norm2``; ``l<i>.mix.y|x|conv|ra|ri`` with ``.b``,
``l<i>.mix.lam|o``; ``l<i>.mix.q|dkv|dkv.norm|uk|uv|g|o``; ``l<i>.mlp.gate|up|down`` or ``l<i>.mlp.router|correction|
e<j>.up|down``; ``final.norm``; ``head``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .duzinex import _NUM, _get
from .gozatar import _positive
from .llama import ConfigError
from .registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MIXERS = ("rglru", "latent_attention")
DECAY_FACTOR = 8.0                # the design fixes the factor of the recurrence gate in the decay's logarithm


@dataclass(frozen=True)
class LuvavikConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    logit_scale: float
    layers: tuple                    # per layer the validated dict {type, mixer, mlp}
    loop: Optional[tuple]            # (start, stop, times) or None
    raw: Optional[dict] = None       # config.json as it was read (written back by ``to_dict``)

    architecture = "Luvavik"

    # ------------------------------------------------------------------ parse
    @classmethod
    def from_dict(cls, d: dict) -> "LuvavikConfig":
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
            mw = where + "mixer."
            if kind == "rglru":
                mixer = dict(width=_positive(m, "width", mw), blocks=_positive(m, "blocks", mw, optional=True) or 1,
                             conv=_positive(m, "conv", mw, optional=True) or 1)
                if mixer["width"] % mixer["blocks"]:
                    raise ConfigError(f"{mw}width {mixer['width']} must be a multiple of blocks {mixer['blocks']}")
            else:
                dim = _positive(m, "dim", mw)
                mixer = dict(heads=_positive(m, "heads", mw), dim=dim, rot_dim=_get(m, "rot_dim", mw, optional=True) or 0,
                             vdim=_positive(m, "vdim", mw, optional=True) or dim, kv_rank=_positive(m, "kv_rank", mw),
                             scale=float(_get(m, "scale", mw, _NUM)), rot_base=None)
                rd = mixer["rot_dim"]
                if rd < 0 or rd % 2:
                    raise ConfigError(f"{mw}rot_dim {rd} must be even and not negative")
                if rd:
                    rot = _get(m, "rot", mw, (dict,))
                    dims = _get(rot, "dims", mw + "rot.", optional=True)
                    if dims is not None and dims != rd:
                        raise ConfigError(f"{mw}rot.dims {dims} must equal rot_dim {rd}")
                    mixer["rot_base"] = float(_get(rot, "base", mw + "rot.", _NUM))
                    if not mixer["rot_base"] > 0:
                        raise ConfigError(f"{mw}rot.base must be positive")
            checked.append(dict(type=kind, mixer=mixer, mlp=cls._mlp(layer.get("mlp"), where + "mlp.")))
        loop = _get(d, "loop", "", (dict,), optional=True)
        span = None
        if loop:
            start, stop, times = (_get(loop, k, "loop.") for k in ("start", "stop", "times"))
            if not (0 <= start < stop <= len(checked)) or times < 1:
                raise ConfigError(f"loop {{start {start}, stop {stop}, times {times}}} does not fit {len(checked)} layers")
            span = (start, stop, times)

        def factor(key):
            v = _get(d, key, "", _NUM, optional=True)
            return float(v) if v is not None else 1.0
        return cls(vocab=_positive(d, "vocab", ""), width=_positive(d, "width", ""),
                   norm_eps=float(_get(d.get("norm") or {}, "eps", "norm.", _NUM)), residual_mult=factor("residual_mult"),
                   logit_scale=factor("logit_scale"), layers=tuple(checked), loop=span, raw=dict(d))

    @staticmethod
    def _mlp(mlp, where: str):
        if mlp is None:
            return None
        kind = _get(mlp, "kind", where, (str,))
        if kind == "dense":
            return dict(kind=kind, ff=_positive(mlp, "ff", where))
        if kind != "moe":
            raise ConfigError(f"config.json field {where}'kind' is {kind!r}; known: 'dense', 'moe'")
        ro = _get(mlp, "router", where, (dict,))
        rw = where + "router."
        out = dict(kind=kind, ff=_positive(_get(mlp, "expert", where, (dict,)), "ff", where + "expert."),
                   experts=_positive(ro, "experts", rw), top=_positive(ro, "top", rw),
                   identity=_get(ro, "identity", rw, optional=True) or 0)
        if out["identity"] < 0 or out["top"] > out["experts"] + out["identity"]:
            raise ConfigError(f"{rw}top {out['top']} cannot be chosen among {out['experts']} experts and {out['identity']} identities")
        return out

    def to_dict(self) -> dict:
        if self.raw is not None:
            return dict(self.raw)
        layers = []
        for l in self.layers:
            m, f = dict(l["mixer"]), l["mlp"]
            if l["type"] == "latent_attention":
                base = m.pop("rot_base")
                if base is not None:
                    m["rot"] = dict(dims=m["rot_dim"], base=base)
            if f is not None and f["kind"] == "moe":
                f = dict(kind="moe", expert=dict(ff=f["ff"]),
                         router=dict(experts=f["experts"], identity=f["identity"], top=f["top"]))
            layers.append(dict(type=l["type"], mixer=m, mlp=f))
        out = dict(architecture=self.architecture, vocab=self.vocab, width=self.width, norm=dict(eps=self.norm_eps),
                   residual_mult=self.residual_mult, logit_scale=self.logit_scale, layers=layers)
        if self.loop:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out

    def stop_token_ids(self) -> list:
        return []

    # ------------------------------------------------------------------ model
    def layer_runs(self) -> list:
        """[(layer, row added in front or None)] in the order the layers run within a step."""
        n = len(self.layers)
        if not self.loop:
            return [(i, None) for i in range(n)]
        start, stop, times = self.loop
        runs = [(i, None) for i in range(start)]
        for p in range(times):
            runs += [(i, p if i == start else None) for i in range(start, stop)]
        return runs + [(i, None) for i in range(stop, n)]

    def to_spec(self) -> ModelSpec:
        W, eps, mult = self.width, self.norm_eps, self.residual_mult

        def norm(name, **kw):
            return PartSpec("rmsnorm", dict(size=W, eps=eps, weight_name="", **kw), prefix=name)

        layers = []
        for i, l in enumerate(self.layers):
            p, m, f = f"l{i}.", l["mixer"], l["mlp"]
            if l["type"] == "rglru":
                mixer = PartSpec("rglru", dict(hidden_size=W, width=m["width"], parts=m["blocks"], taps=m["conv"],
                                               decay_factor=DECAY_FACTOR, out_scale=mult), prefix=p + "mix.")
            else:
                rope = PartSpec("rotary", dict(theta=m["rot_base"], rotary_dim=m["rot_dim"])) if m["rot_dim"] else None
                mixer = PartSpec("rotary_latent_attention", dict(
                    hidden_size=W, num_heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], v_head_dim=m["vdim"],
                    kv_rank=m["kv_rank"], scale=m["scale"], eps=eps, position=rope, gate="element", out_scale=mult),
                    prefix=p + "mix.")
            ffn, norms = None, {"mixer": norm(p + "norm1")}
            if f is not None:
                norms["ffn"] = norm(p + "norm2")
                if f["kind"] == "dense":
                    ffn = PartSpec("geglu", dict(hidden_size=W, intermediate_size=f["ff"], out_scale=mult,
                                                 names=dict(gate="gate", up="up", down="down")), prefix=p + "mlp.")
                else:
                    ffn = PartSpec("routed_experts", dict(
                        hidden_size=W, intermediate_size=f["ff"], experts=f["experts"], top=f["top"], identity=f["identity"],
                        activation="relu2", score="softmax", normalize=False, weight_scale=mult), prefix=p + "mlp.")
            layers.append(LayerSpec(block="prenorm", mixer=mixer, ffn=ffn, norms=norms))
        schedule = tuple(ScheduleEntry(layer, run, True, adds_row=row) for run, (layer, row) in enumerate(self.layer_runs()))
        rows = None
        if self.loop:
            rows = PartSpec("row_table", dict(rows=self.loop[2], hidden_size=W, weight_name="loop.step"))
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=W,
            embedding=PartSpec("embedding", dict(vocab_size=self.vocab, hidden_size=W, weight_name="embed")),
            layers=tuple(layers), schedule=schedule, pass_rows=rows,
            final_norm=norm("final.norm", weight_scale=self.logit_scale),       # the head is linear: its factor rides in the norm
            head=PartSpec("lm_head", dict(vocab_size=self.vocab, hidden_size=W, weight_name="head")),
            max_position=0)
        spec.validate()
        return spec


register_architecture(LuvavikConfig.architecture, LuvavikConfig)
