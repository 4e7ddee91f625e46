"""Causal grouped-query attention with a gate on its output, as a mixer (not in the reference).

    q = Wq x (+ bq),  k = Wk x (+ bk),  v = Wv x (+ bv)          per head: q, k of size dim, v of size vdim
    q_t ← q_t · (1 + coef · ln(⌊(t + 1) / every⌋ + 1))            (``q_temp``: the query grows with its position t)
    q, k ← q, k / sqrt(mean(·²) + eps) ⊙ w per head               (``qk_norm_eps``: w of size dim, one for q and one for k)
    rotation over the first dims of q and k                        (``position``: neighbouring pairs, pairing "interleaved",
                                                                    or dim i with dim i + r/2, pairing "half")
    s_h(i, j) = (q_i,h · k_j,g(h)) · scale + R[row(i − j), h]     (``distance_rows`` rows of a learned table R; the scale
                                                                    does not multiply it)
    p_h(i, j) = e^{s} / (Σ_j e^{s} (+ e^{sink_h}))                 over the visible j ≤ i (``window`` w: i − j < w);
                                                                    ``sink``: a learned score per head, no key, no value
    y += Wo · concat_h( gate ⊙ Σ_j p_h(i, j) v_j,g(h) )           gate: sigmoid(w_g,h · x) per head (``gate`` "head"),
                                                                    sigmoid(Wg x) per element ("element"), or none (None)

Rows of the distance table, for B rows and the distance ``distance_far`` = D at which the last row is reached: distances
n < B/2 have a row each; n ≥ B/2 takes row min(B − 1, B/2 + ⌊ln(n / (B/2)) / ln(D / (B/2)) · (B − B/2)⌋). When the weights
are bound the table is spread out by distance once, [heads, distances up to the first that takes the last row], so
that the attention kernels look a score up by min(i − j, last).

``shares_kv``: the mixer has no tensors of keys and values and reads the rows that another layer's run of the same step
has cached (as they stand there, normed and rotated), with queries of its own.

Every option is a constructor parameter. The projections of q, k, v and the gates run as ONE product over the stacked
weight; one kernel then adds the biases, applies query factor or norms and the rotation, writes q and the cache rows and
hands the gates' arguments on. Scores, softmax, norms, gates, angles and the factor are 32-bit in every mode.
"""
from __future__ import annotations

import math

import torch

from ..csrc import lib as K
from .attention import attend_paged, attention_modules
from .base import KVCacheRequest, Mixer, WeightSpec
from .linear import Linear
from .registry import build_part, register_part
from ..phases import phase


def distance_row(n: int, rows: int, far: float) -> int:
    """The row of a table of ``rows`` rows that the distance ``n`` takes (see the module's text)."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))


def distance_table(rel: torch.Tensor, far: float) -> torch.Tensor:
    """``rel`` [rows, heads] -> float32 [heads, distances]: entry n is the row that distance n takes; the last entry
    stands for every larger distance."""
    rows = rel.shape[0]
    picks, n = [], 0
    while True:
        r = distance_row(n, rows, far)
        picks.append(r)
        if r >= rows - 1 or n > (1 << 22):
            break
        n += 1
    idx = torch.tensor(picks, dtype=torch.long, device=rel.device)
    return rel.float().index_select(0, idx).t().contiguous()


@register_part("mixer", "gated_attention")
class GatedAttention(Mixer):
    graph_safe = True
    kernel_modules = ("sandwich",)

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, v_head_dim: int, scale: float,
                 bias: bool = False, q_temp: tuple | None = None, distance_rows: int = 0, distance_far: float = 0.0,
                 position=None, sink: bool = False, window=None, gate: str | None = "head", qk_norm_eps: float | None = None,
                 shares_kv: bool = False, prefix: str = "", names: dict | None = None):
        super().__init__(prefix)
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads are no multiple of {num_kv_heads} kv heads")
        self.hidden_size, self.num_heads, self.num_kv_heads = int(hidden_size), int(num_heads), int(num_kv_heads)
        self.head_dim, self.v_head_dim, self.scale = int(head_dim), int(v_head_dim), float(scale)
        self.bias, self.has_sink = bool(bias), bool(sink)
        self.q_temp = (float(q_temp[0]), int(q_temp[1])) if q_temp else None          # (coef, every)
        # rows of the distance table; negative −n: the checkpoint's tensor decides (random weights take n)
        self.distance_rows, self.distance_far = int(distance_rows), float(distance_far)
        self.window = int(window) if window else None
        if gate not in (None, "head", "element"):
            raise ValueError(f"{prefix}: a gate is per 'head', per 'element' or None, got {gate!r}")
        self.gate, self.shares_kv = gate, bool(shares_kv)
        self.qk_norm_eps = None if qk_norm_eps is None else float(qk_norm_eps)
        n = dict(q="q", k="k", v="v", g="g", o="o", rel="rel", sink="sink", bias_suffix=".b", norm_suffix=".norm")
        n.update(names or {})
        self.bias_suffix, self.norm_suffix = n.pop("bias_suffix"), n.pop("norm_suffix")
        self.names = {k: prefix + v for k, v in n.items()}
        self.position = build_part("position", position) if position is not None else None
        self.halves = self.position is not None and getattr(self.position, "pairing", "half") == "half"
        # which kernel places q, k and v: the one with the query factor and the head gates, or the one with the heads' norms
        self.plain_store = not self.halves and self.qk_norm_eps is None and gate == "head" and not self.shares_kv
        if not self.plain_store and self.q_temp:
            raise ValueError(f"{prefix}: the query factor goes with neighbouring pairs, a gate per head and heads without a norm")
        if gate == "head" and not self.plain_store:
            raise ValueError(f"{prefix}: a gate per head goes with neighbouring pairs and heads without a norm")
        self.kernel_modules_bf16 = attention_modules(self.head_dim, self.v_head_dim)
        self.proj = self.o = self.qkv_bias = self.sink = self.dist = self.q_norm = self.k_norm = None

    def children(self):
        return [self.position] if self.position is not None else []

    def _shapes(self):
        W, nh, g, d, vd = self.hidden_size, self.num_heads, self.num_kv_heads, self.head_dim, self.v_head_dim
        return dict(q=(nh * d, W)) if self.shares_kv else dict(q=(nh * d, W), k=(g * d, W), v=(g * vd, W))

    def weight_specs(self):
        W, nh, vd = self.hidden_size, self.num_heads, self.v_head_dim
        specs = [WeightSpec(self.names[k], s) for k, s in self._shapes().items()]
        specs.append(WeightSpec(self.names["o"], (W, nh * vd)))
        if self.gate:
            specs.append(WeightSpec(self.names["g"], (nh if self.gate == "head" else nh * vd, W)))
        if self.qk_norm_eps is not None:
            specs += [WeightSpec(self.names[k] + self.norm_suffix, (self.head_dim,), init="ones") for k in ("q", "k") if k in self._shapes()]
        if self.bias:
            specs += [WeightSpec(self.names[k] + self.bias_suffix, (s[0],)) for k, s in self._shapes().items()]
        if self.distance_rows:
            specs.append(WeightSpec(self.names["rel"], (self.distance_rows, nh)))
        if self.has_sink:
            specs.append(WeightSpec(self.names["sink"], (nh,)))
        return specs

    def cache_request(self):
        vd = self.v_head_dim if self.v_head_dim != self.head_dim else None
        return KVCacheRequest(self.num_kv_heads, self.head_dim, self.window, v_head_dim=vd)

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        own = list(self._shapes())
        parts = [tensors[self.names[k]] for k in own + (["g"] if self.gate else [])]
        if len({p.dtype for p in parts}) != 1:
            raise ValueError(f"{self.prefix}: the projections of q, k, v and the gates must share a storage type")
        self.proj = Linear(torch.cat(parts, dim=0))
        self.o = Linear(tensors[self.names["o"]])
        if self.bias:
            self.qkv_bias = torch.cat([tensors[self.names[k] + self.bias_suffix] for k in own]).contiguous()
        if self.qk_norm_eps is not None:
            self.q_norm = tensors[self.names["q"] + self.norm_suffix].contiguous()
            self.k_norm = None if self.shares_kv else tensors[self.names["k"] + self.norm_suffix].contiguous()
        self.sink = tensors[self.names["sink"]].float().contiguous() if self.has_sink else None        # a score: 32-bit
        self.dist = None
        if self.distance_rows:
            rel = tensors[self.names["rel"]]
            if rel.shape[0] < 2 or not self.distance_far > rel.shape[0] // 2:
                raise ValueError(f"{self.prefix}: a distance table of {rel.shape[0]} rows and a last row reached at "
                                 f"{self.distance_far} do not fit together")
            self.dist = distance_table(rel, self.distance_far)
        # arrival counters of the split-key decode attention; the kernel returns them to zero
        self.counters = torch.zeros(4096, dtype=torch.int32, device=rt.device)

    def forward(self, x, step, cache, residual):
        nh, g, d, vd = self.num_heads, self.num_kv_heads, self.head_dim, self.v_head_dim
        T, dev, act = x.shape[0], x.device, self.rt.act_dtype
        freq, rd, amp = None, 0, 1.0
        if self.position is not None:
            freq, rd = self.position.rotary()
            amp = getattr(self.position, "amplitude", 1.0)
        with phase("qkv_projection_ms"):
            proj = self.proj(x, out_dtype=torch.float32)            # biases, factor and rotation read unrounded products
        if cache.writes == self.shares_kv and (self.shares_kv or not self.plain_store):
            raise ValueError(f"{self.prefix}: a layer without k/v projections reads another run's cache, any other writes its own")
        kv = 0 if self.shares_kv else g
        with phase("rotary+kv_append_ms"):
            q = torch.empty(T, nh * d, dtype=act, device=dev)
            if self.plain_store:
                gates = torch.empty(T, nh, dtype=torch.float32, device=dev)
                coef, every = self.q_temp or (0.0, 1)
                K.gated_qkv_store(proj, self.qkv_bias, q, cache.k_pool, cache.v_pool, cache, gates, freq, nh, g, d, vd, rd,
                                  write_kv=cache.writes, rot_mult=amp, temp_coef=coef, temp_every=every)
            else:
                K.qkv_norm_rot_store(proj, self.qkv_bias, q, cache.k_pool, cache.v_pool, cache, freq, nh, kv, d, vd, rd,
                                     q_weight=self.q_norm, k_weight=self.k_norm, eps=self.qk_norm_eps or 0.0, rot_mult=amp,
                                     halves=self.halves)
        with phase("distance_attention_ms" if self.dist is not None else "attention_ms"):
            ctx = self.attend(q, step, cache)
        if self.gate == "head":
            with phase("head_gate_ms"):
                K.scale_rows_sigmoid(ctx.view(T * nh, vd), gates.view(T * nh))
        elif self.gate == "element":
            with phase("element_gate_ms"):
                K.gate_elements(ctx, proj[:, nh * d + kv * (d + vd):])
        with phase("o_projection+attention_residual_ms"):
            self.o(ctx, out=residual, accumulate=True)

    def attend(self, q, step, cache):
        """The heads' outputs [T, heads·vdim] over the cached keys and values, the step's own included."""
        return attend_paged(q, step, cache, self.num_heads, self.num_kv_heads, self.head_dim, self.window, self.scale, self.sink,
                            self.counters, dist_bias=self.dist, vd=self.v_head_dim)
