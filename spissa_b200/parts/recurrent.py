"""Mixers that carry a fixed-size state instead of keys and values (not in the reference).

Retention: linear attention with one fixed decay per head and neither softmax nor denominator.
    q, k [heads·dim], v, g [heads·vdim] = projections of x (no bias);  per head, with S₀ = 0 [dim, vdim]:
    S_t = γ_h · S_{t-1} + (k_t / √dim) v_tᵀ,   o_t = S_tᵀ q_t,   ô_t = o_t / sqrt(mean(o_t²) + eps);
    y_t = Wo · ( concat_h(ô_t) ⊙ silu(g_t) ).

minGRU: a gated recurrence whose gates read the current token only.
    z_t = sigmoid(Wz x_t + bz),  u_t = Wx x_t + bx,  c_t = u_t + ½ where u_t ≥ 0 and sigmoid(u_t) where u_t < 0;
    S_t = (1 − z_t) ⊙ S_{t-1} + z_t ⊙ c_t  (S₀ = 0),   y_t = Wo · ( S_t ⊙ silu(Wg x_t) ).

Gated linear attention: linear attention whose state decays per key channel by a gate that reads the token.
    q, k [heads·dim], v, g [heads·vdim] = projections of x (no bias), q times dim^(−1/2);
    z = Wa2 (Wa1 x) + b [heads·dim] through a low rank,  α_t = sigmoid(z_t)^(1/τ);  per head, with S₀ = 0 [dim, vdim]:
    S_t = diag(α_t) S_{t-1} + k_t v_tᵀ,   o_t = S_tᵀ q_t,   ô_t = o_t / sqrt(mean(o_t²) + eps) ⊙ w  (w [vdim], shared by heads);
    y_t = Wo · ( concat_h(ô_t) ⊙ silu(g_t) ) · out_scale.

RG-LRU block (Griffin's recurrent block): a real-gated linear recurrent unit behind a short causal convolution, times a
gelu branch, both of size ``width``:
    y_t = gelu(Wy x_t + by),  u_t = conv(Wx x_t + bx)  (per channel, ``taps`` taps, bias; the inputs before the start are 0);
    u is cut into ``parts`` equal parts with square gate matrices:  r = sigmoid(Ra u + ρ),  i = sigmoid(Ri u + ι);
    log a_t = −decay_factor · r ⊙ softplus(λ),  S_t = a_t ⊙ S_{t-1} + sqrt(1 − a_t²) ⊙ i ⊙ u_t  (S₀ = 0);
    y += Wo (S_t ⊙ y_t) · out_scale.
The convolution's last inputs are a second state, a ring of ``taps`` rows (row p mod taps holds position p's input).

mLSTM (the matrix memory of xLSTM): linear attention with an exponential input gate, a forget gate and a normaliser.
    q, k [heads·dim], v, g [heads·vdim] = projections of x (no bias), q times dim^(−1/2);  per head, with c = gate_cap:
    i = c·tanh((Wi x + bi) / c),  f = ln sigmoid(c·tanh((Wf x + bf) / c));  m_t = max(f + m_{t-1}, i)  (m₀ = 0);
    S_t = e^{f + m_{t-1} − m_t} S_{t-1} + e^{i − m_t} k vᵀ,  n_t likewise with k alone  (S₀ = 0, n₀ = 0);
    o = S_tᵀ q / (max(|n_t · q|, e^{−m_t}) + 1e-6),  ô = o / sqrt(mean(o²) + eps) per head;
    y_t = Wo · ( concat_h(ô) ⊙ w ⊙ sigmoid(g) )   (w over all heads).

All states are 32-bit and belong to the sequence's slot; the recurrences run in 32-bit on the unrounded
projections, which are one matrix product over the stacked weights.
"""
from __future__ import annotations

import torch

from ..csrc import lib as K
from .base import CacheBundle, Mixer, StateRequest, WeightSpec
from .linear import Linear
from .registry import register_part
from ..phases import phase


@register_part("mixer", "retention")
class Retention(Mixer):
    graph_safe = True
    kernel_modules = ("seqmix",)

    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, decay, eps: float, prefix: str = "",
                 names: dict | None = None):
        super().__init__(prefix)
        self.hidden_size, self.num_heads, self.dim, self.vdim = int(hidden_size), int(num_heads), int(dim), int(vdim)
        self.decay_values = [float(g) for g in decay]
        if len(self.decay_values) != self.num_heads:
            raise ValueError(f"{prefix}: {len(self.decay_values)} decays for {self.num_heads} heads")
        self.eps = float(eps)
        n = dict(q="q", k="k", v="v", g="g", o="o")
        n.update(names or {})
        self.names = {k: prefix + v for k, v in n.items()}
        self.proj = self.o = self.decay = None

    def weight_specs(self):
        H, nh, d, vd = self.hidden_size, self.num_heads, self.dim, self.vdim
        return [WeightSpec(self.names["q"], (nh * d, H)), WeightSpec(self.names["k"], (nh * d, H)),
                WeightSpec(self.names["v"], (nh * vd, H)), WeightSpec(self.names["g"], (nh * vd, H)),
                WeightSpec(self.names["o"], (H, nh * vd))]

    def cache_request(self):
        return StateRequest((self.num_heads, self.dim, self.vdim), torch.float32)

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        self.proj = Linear(torch.cat([tensors[self.names[k]] for k in ("q", "k", "v", "g")], dim=0))
        self.o = Linear(tensors[self.names["o"]])
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=rt.device)

    def forward(self, x, step, cache, residual):
        with phase("mixer_projection_ms"):
            p = self.proj(x, out_dtype=torch.float32)
        with phase("retention_ms"):
            y = torch.empty(x.shape[0], self.num_heads * self.vdim, dtype=self.rt.act_dtype, device=x.device)
            K.retention(p, cache.state, self.decay, y, step, self.num_heads, self.dim, self.vdim, self.eps)
        with phase("o_projection+mixer_residual_ms"):
            self.o(y, out=residual, accumulate=True)


@register_part("mixer", "mingru")
class MinGRU(Mixer):
    graph_safe = True
    kernel_modules = ("seqmix",)

    def __init__(self, hidden_size: int, width: int, prefix: str = "", names: dict | None = None):
        super().__init__(prefix)
        self.hidden_size, self.width = int(hidden_size), int(width)
        n = dict(z="z", zb="z.b", x="x", xb="x.b", g="g", o="o")
        n.update(names or {})
        self.names = {k: prefix + v for k, v in n.items()}
        self.proj = self.o = self.zb = self.xb = None

    def weight_specs(self):
        H, W = self.hidden_size, self.width
        return [WeightSpec(self.names["z"], (W, H)), WeightSpec(self.names["zb"], (W,)),
                WeightSpec(self.names["x"], (W, H)), WeightSpec(self.names["xb"], (W,)),
                WeightSpec(self.names["g"], (W, H)), WeightSpec(self.names["o"], (H, W))]

    def cache_request(self):
        return StateRequest((self.width,), torch.float32)

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        self.proj = Linear(torch.cat([tensors[self.names[k]] for k in ("z", "x", "g")], dim=0))
        self.o = Linear(tensors[self.names["o"]])
        self.zb = tensors[self.names["zb"]].contiguous()
        self.xb = tensors[self.names["xb"]].contiguous()

    def forward(self, x, step, cache, residual):
        with phase("mixer_projection_ms"):
            p = self.proj(x, out_dtype=torch.float32)
        with phase("mingru_ms"):
            y = torch.empty(x.shape[0], self.width, dtype=self.rt.act_dtype, device=x.device)
            K.mingru(p, self.zb, self.xb, cache.state, y, step, self.width)
        with phase("o_projection+mixer_residual_ms"):
            self.o(y, out=residual, accumulate=True)


@register_part("mixer", "gla")
class GatedLinearAttention(Mixer):
    """``rank`` is the size of the low-rank input of the decays; None: the checkpoint's tensors say it (random weights
    then take 16)."""
    graph_safe = True
    kernel_modules = ("hybrid",)

    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, tau: float, eps: float,
                 rank: int | None = None, out_scale: float = 1.0, prefix: str = "", names: dict | None = None):
        super().__init__(prefix)
        self.hidden_size, self.num_heads, self.dim, self.vdim = int(hidden_size), int(num_heads), int(dim), int(vdim)
        self.tau, self.eps, self.out_scale = float(tau), float(eps), float(out_scale)
        if not self.tau > 0:
            raise ValueError(f"{prefix}: tau must be positive")
        self.rank = int(rank) if rank else None
        n = dict(q="q", k="k", v="v", g="g", o="o", a1="a1", a2="a2", a2b="a2.b", norm="norm")
        n.update(names or {})
        self.names = {k: prefix + v for k, v in n.items()}
        self.proj = self.o = self.a2 = self.a2b = self.norm = None

    def weight_specs(self):
        H, nh, d, vd, r = self.hidden_size, self.num_heads, self.dim, self.vdim, self.rank or -16
        return [WeightSpec(self.names["q"], (nh * d, H)), WeightSpec(self.names["k"], (nh * d, H)),
                WeightSpec(self.names["v"], (nh * vd, H)), WeightSpec(self.names["g"], (nh * vd, H)),
                WeightSpec(self.names["o"], (H, nh * vd)), WeightSpec(self.names["a1"], (r, H)),
                WeightSpec(self.names["a2"], (nh * d, r)), WeightSpec(self.names["a2b"], (nh * d,)),
                WeightSpec(self.names["norm"], (vd,), init="ones")]

    def cache_request(self):
        return StateRequest((self.num_heads, self.dim, self.vdim), torch.float32)

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        a1, a2 = tensors[self.names["a1"]], tensors[self.names["a2"]]
        if a1.shape[0] != a2.shape[1]:
            raise ValueError(f"{self.prefix}: the two halves of the decay projection disagree on the rank "
                             f"({a1.shape[0]} and {a2.shape[1]})")
        self.rank = int(a1.shape[0])
        self.proj = Linear(torch.cat([tensors[self.names[k]] for k in ("q", "k", "v", "g", "a1")], dim=0))
        self.o = Linear(tensors[self.names["o"]])
        self.a2 = a2.contiguous()
        self.a2b = tensors[self.names["a2b"]].contiguous()
        self.norm = tensors[self.names["norm"]].contiguous()

    def forward(self, x, step, cache, residual):
        with phase("mixer_projection_ms"):
            p = self.proj(x, out_dtype=torch.float32)              # the recurrence reads unrounded products
        with phase("gla_ms"):
            y = torch.empty(x.shape[0], self.num_heads * self.vdim, dtype=self.rt.act_dtype, device=x.device)
            K.gla(p, cache.state, self.a2, self.a2b, self.norm, y, step, self.num_heads, self.dim, self.vdim, self.rank,
                  self.tau, self.eps, self.out_scale)
        with phase("o_projection+mixer_residual_ms"):
            self.o(y, out=residual, accumulate=True)


@register_part("mixer", "rglru")
class RGLRU(Mixer):
    """``out_scale``: a factor on the mixer's output, applied to the 32-bit product S ⊙ y in front of the output projection."""
    graph_safe = True
    kernel_modules = ("rglru",)

    def __init__(self, hidden_size: int, width: int, parts: int, taps: int, decay_factor: float = 8.0, out_scale: float = 1.0,
                 prefix: str = "", names: dict | None = None):
        super().__init__(prefix)
        self.hidden_size, self.width, self.parts, self.taps = int(hidden_size), int(width), int(parts), int(taps)
        self.decay_factor, self.out_scale = float(decay_factor), float(out_scale)
        if self.parts < 1 or self.width % self.parts:
            raise ValueError(f"{prefix}: a width of {self.width} is not {self.parts} equal parts")
        if self.taps < 1:
            raise ValueError(f"{prefix}: the convolution needs at least one tap")
        n = dict(y="y", yb="y.b", x="x", xb="x.b", conv="conv", convb="conv.b", ra="ra", rab="ra.b", ri="ri", rib="ri.b",
                 lam="lam", o="o")
        n.update(names or {})
        self.names = {k: prefix + v for k, v in n.items()}
        self.proj = self.o = self.w = None

    def weight_specs(self):
        H, W, P, s, n = self.hidden_size, self.width, self.parts, self.width // self.parts, self.names
        return [WeightSpec(n["y"], (W, H)), WeightSpec(n["yb"], (W,)), WeightSpec(n["x"], (W, H)), WeightSpec(n["xb"], (W,)),
                WeightSpec(n["conv"], (W, self.taps)), WeightSpec(n["convb"], (W,)),
                WeightSpec(n["ra"], (P, s, s)), WeightSpec(n["rab"], (P, s)), WeightSpec(n["ri"], (P, s, s)),
                WeightSpec(n["rib"], (P, s)), WeightSpec(n["lam"], (W,)), WeightSpec(n["o"], (H, W))]

    def cache_request(self):
        ring = StateRequest((self.taps, self.width), torch.float32) if self.taps > 1 else None
        return CacheBundle.of(conv=ring, state=StateRequest((self.width,), torch.float32))

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        n = self.names
        if tensors[n["y"]].dtype != tensors[n["x"]].dtype:
            raise ValueError(f"{self.prefix}: the projections of one input must share a storage type")
        self.proj = Linear(torch.cat([tensors[n["y"]], tensors[n["x"]]], dim=0))
        self.o = Linear(tensors[n["o"]])
        small = {k: tensors[n[k]].float().reshape(-1).contiguous() for k in ("yb", "xb", "convb", "rab", "rib")}
        # ln(1 + e^λ) in 64-bit, rounded once
        decay = (self.decay_factor * torch.logaddexp(tensors[n["lam"]].double(), torch.zeros((), dtype=torch.float64, device=rt.device)))
        self.w = dict(small, conv=tensors[n["conv"]].float().contiguous(), decay=decay.float().contiguous(),
                      ra=tensors[n["ra"]].contiguous(), ri=tensors[n["ri"]].contiguous())

    def forward(self, x, step, cache, residual):
        with phase("mixer_projection_ms"):
            p = self.proj(x, out_dtype=torch.float32)              # the recurrence reads unrounded products
        with phase("rglru_ms"):
            y = torch.empty(x.shape[0], self.width, dtype=self.rt.act_dtype, device=x.device)
            ring = cache.get("conv")
            K.rglru(p, self.w, ring.state if ring is not None else None, cache["state"].state, y, step, self.width, self.taps,
                    self.parts, self.out_scale)
        with phase("o_projection+mixer_residual_ms"):
            self.o(y, out=residual, accumulate=True)


@register_part("mixer", "mlstm")
class MLSTM(Mixer):
    graph_safe = True
    kernel_modules = ("mlstm",)

    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, gate_cap: float, eps: float, prefix: str = "",
                 names: dict | None = None):
        super().__init__(prefix)
        self.hidden_size, self.num_heads, self.dim, self.vdim = int(hidden_size), int(num_heads), int(dim), int(vdim)
        self.gate_cap, self.eps = float(gate_cap), float(eps)
        if not self.gate_cap > 0:
            raise ValueError(f"{prefix}: the cap of the gates must be positive")
        n = dict(q="q", k="k", v="v", g="g", o="o", i="i", ib="i.b", f="f", fb="f.b", norm="norm")
        n.update(names or {})
        self.names = {k: prefix + v for k, v in n.items()}
        self.proj = self.o = self.w = None

    def weight_specs(self):
        H, nh, d, vd, n = self.hidden_size, self.num_heads, self.dim, self.vdim, self.names
        return [WeightSpec(n["q"], (nh * d, H)), WeightSpec(n["k"], (nh * d, H)), WeightSpec(n["v"], (nh * vd, H)),
                WeightSpec(n["g"], (nh * vd, H)), WeightSpec(n["o"], (H, nh * vd)), WeightSpec(n["norm"], (nh * vd,), init="ones"),
                WeightSpec(n["i"], (nh, H)), WeightSpec(n["ib"], (nh,)), WeightSpec(n["f"], (nh, H)), WeightSpec(n["fb"], (nh,))]

    def cache_request(self):
        return CacheBundle.of(state=StateRequest((self.num_heads, self.dim, self.vdim), torch.float32),
                              nm=StateRequest((self.num_heads, self.dim + 1), torch.float32))

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        n = self.names
        parts = [tensors[n[k]] for k in ("q", "k", "v", "g", "i", "f")]
        if len({p.dtype for p in parts}) != 1:
            raise ValueError(f"{self.prefix}: the projections of one input must share a storage type")
        rows = sum(p.shape[0] for p in parts)
        if rows % 4:                                     # the kernels' 16-byte pieces want rows of a multiple of four numbers
            parts.append(torch.zeros(4 - rows % 4, self.hidden_size, dtype=parts[0].dtype, device=parts[0].device))
        self.proj = Linear(torch.cat(parts, dim=0))
        self.o = Linear(tensors[n["o"]])
        self.w = {k: tensors[n[k]].float().contiguous() for k in ("ib", "fb", "norm")}

    def forward(self, x, step, cache, residual):
        with phase("mixer_projection_ms"):
            p = self.proj(x, out_dtype=torch.float32)              # the gates and the memory read unrounded products
        with phase("mlstm_ms"):
            y = torch.empty(x.shape[0], self.num_heads * self.vdim, dtype=self.rt.act_dtype, device=x.device)
            K.mlstm(p, self.w, cache["state"].state, cache["nm"].state, y, step, self.num_heads, self.dim, self.vdim,
                    self.gate_cap, self.eps)
        with phase("o_projection+mixer_residual_ms"):
            self.o(y, out=residual, accumulate=True)
