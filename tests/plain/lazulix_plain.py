"""Plain, slow implementation of the Lazulix decoder: whole sequences, no cache, no state carried between calls.

One function per mechanism, plain tensor arithmetic on the CPU (float64 unless told otherwise). It shares no code
with ``spissa_b200``: it reads config.json keys and a dict of tensors by their checkpoint names. Notation: x is the
residual stream [T, W], n(·; w) a layer norm with a weight and no bias, r(·) a weightless RMS norm, σ the logistic function.

    embedding       x_t = E[id_t] · scale
    layer           x ← x + n(mixer(n(x; w1)); w1b);   x ← x + n(ff(n(x; w2)); w2b)      (the second only with an ``mlp``)
    mlstm           C_t = e^{f_t} C_{t−1} + e^{i_t} k_t v_tᵀ and its normaliser, kept times e^{−m_t} with a running
                    maximum m that starts at 0; gates i = c tanh(ĩ/c), f = ln σ(c tanh(f̃/c));
                    out = O (r(o) ⊙ w ⊙ σ(G a))
    attention       biased q, k, v; (``attention_2``: weighted RMS norm of q and k per head;) rotation by halves with
                    frequencies interpolated pair by pair; softmax over all earlier keys; (``attention_2``: the
                    concatenated heads ⊙ σ(G a), and perhaps another layer's keys and values)
    feed-forward    g = min(Gt a, L), u = clamp(Up a, ±L):  Dn (g σ(1.702 g) (u + 1))
    head            logits = n(x; w_f) · Eᵀ
"""
from __future__ import annotations

import math

import torch

GATE_SLOPE = 1.702


def layer_norm(x, w, eps):
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * w


def rms_norm(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def capped_gates(a, w, p, cap):
    """(input gate, forget gate) as logarithms, [T, heads] each."""
    i = cap * torch.tanh((a @ w[p + "i"].T + w[p + "i.b"]) / cap)
    z = cap * torch.tanh((a @ w[p + "f"].T + w[p + "f.b"]) / cap)
    return i, -torch.log1p(torch.exp(-z))


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, d], v [T, H, vd], gate logarithms [T, H] -> (outputs [T, H, vd], S, n, m after the last token)."""
    T, H, d = q.shape
    vd = v.shape[-1]
    out = torch.zeros(T, H, vd, dtype=q.dtype)
    S, n, m = torch.zeros(H, d, vd, dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        m = new
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        over = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(dim=1) / over[:, None]
    return out, S, n, m


def mlstm(a, w, p, mx, eps):
    """Mixer 'mlstm'."""
    T, H, d, vd = a.shape[0], mx["heads"], mx["dim"], mx["vdim"]
    q = (a @ w[p + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (a @ w[p + "k"].T).reshape(T, H, d)
    v = (a @ w[p + "v"].T).reshape(T, H, vd)
    i, f = capped_gates(a, w, p, mx["gate_cap"])
    o = rms_norm(matrix_memory(q, k, v, i, f)[0], eps).reshape(T, H * vd)
    return (o * w[p + "norm"] * torch.sigmoid(a @ w[p + "g"].T)) @ w[p + "o"].T


def pair_frequencies(rot):
    """Angle per position of every pair, and the factor of cos and sin."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def place(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(place(sc["fast"])), 0), min(math.ceil(place(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = (i - lo) / max(hi - lo, 0.001)
        r = 0.0 if r < 0 else 1.0 if r > 1 else r
        out.append(fi / sc["factor"] * r + fi * (1.0 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(v, rot):
    """v [T, heads, dim]: dim i < dims/2 pairs with dim i + dims/2; dims beyond ``dims`` pass."""
    if not rot:
        return v
    T, dims = v.shape[0], rot["dims"]
    half = dims // 2
    freq, amp = pair_frequencies(rot)
    ang = torch.arange(T, dtype=torch.float64)[:, None] * torch.tensor(freq, dtype=torch.float64)[None, :]
    c, s = (torch.cos(ang) * amp).to(v.dtype)[:, None, :], (torch.sin(ang) * amp).to(v.dtype)[:, None, :]
    lo, hi, rest = v[..., :half], v[..., half:dims], v[..., dims:]
    return torch.cat([lo * c - hi * s, hi * c + lo * s, rest], dim=-1)


def causal_mix(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, vd] -> [T, H, vd]; query head h reads key/value head floor(h / (H/G))."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], -math.inf)
        e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
        out.append((e / e.sum(dim=-1, keepdim=True)) @ v[:, g])
    return torch.stack(out, dim=1)


def attention(a, w, p, mx, eps, kind="attention", kept=None):
    """Mixers 'attention' and 'attention_2'; ``kept``: keys and values by layer, this layer's own are added under
    ``kept["own"]``."""
    T, H, G, d, vd = a.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    normed = kind == "attention_2"

    def heads(name, n):
        return (a @ w[p + name].T + w[p + name + ".b"]).reshape(T, n, -1)

    def placed(x, name):
        if normed:
            x = rms_norm(x, eps) * w[p + name + ".norm"]
        return rotate_halves(x, mx.get("rot"))
    q = placed(heads("q", H), "q")
    if mx.get("kv_from") is None:
        k, v = placed(heads("k", G), "k"), heads("v", G)
    else:
        k, v = kept[mx["kv_from"]]
    if kept is not None:
        kept["own"] = (k, v)
    o = causal_mix(q, k, v, mx["scale"]).reshape(T, H * vd)
    if normed:
        o = o * torch.sigmoid(a @ w[p + "g"].T)
    return o @ w[p + "o"].T


def clamped_unit(a, w, p, limit):
    g = torch.clamp(a @ w[p + "gate"].T, max=limit)
    u = torch.clamp(a @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(GATE_SLOPE * g) * (u + 1.0)) @ w[p + "down"].T


def forward(cfg: dict, weights: dict, ids, dtype=torch.float64, layers_out: list | None = None):
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(ids, dtype=torch.long)] * cfg["embedding"]["scale"]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        a = layer_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "mlstm":
            y = mlstm(a, w, p + "mix.", mx, eps)
        elif layer["type"] in ("attention", "attention_2"):
            y = attention(a, w, p + "mix.", mx, eps, layer["type"], kept)
            kept[i] = kept.pop("own")
        else:
            raise ValueError(f"unknown layer type {layer['type']!r}")
        x = x + layer_norm(y, w[p + "norm1b"], eps)
        f = layer.get("mlp")
        if f is not None:
            y = clamped_unit(layer_norm(x, w[p + "norm2"], eps), w, p + "mlp.", f["limit"])
            x = x + layer_norm(y, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["embed"].T


def generate_greedy(cfg, weights, prompt, n_new: int) -> list:
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(torch.argmax(forward(cfg, weights, ids)[-1])))
    return ids[len(prompt):]
