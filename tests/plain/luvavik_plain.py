"""Plain, slow implementation of the Luvavik decoder: whole sequences, no cache, no state carried between calls.

One function per mechanism, plain tensor arithmetic on the CPU (float64 unless told otherwise). It shares no code
with ``spissa_b200``: it reads config.json keys and a dict of tensors by their checkpoint names. Notation: x is the
residual stream [T, W], m the residual multiplier, n(·; w) an RMS norm with a plain weight, σ the logistic function.

    embedding       x_t = E[id_t]
    passes          layers start … stop−1 run ``times`` times in a row; in front of pass p a learned row L[p] joins x
    layer           x ← x + m · mixer(n(x; w1));   x ← x + m · ff(n(x; w2))
    rglru           y = gelu(A a + α), u = conv(B a + β); gates from u part by part; S_t = d_t S_{t−1} + sqrt(1 − d_t²) i_t u_t;
                    out = O (S ⊙ y)
    latent attn.    keys and values are images of a normed low-rank row, plus one rotated key part shared by all heads;
                    the concatenated heads times σ(G a), element by element
    feed-forward    gelu-gated, or routed experts (squared relu, no gate) with experts that return their input
    head            logits = (n(x; w_f) · Hᵀ) · logit_scale
"""
from __future__ import annotations

import math

import torch

DECAY_FACTOR = 8.0


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(z, taps, bias):
    """z [T, C]; taps [C, n], the last one the current token's; nothing before the first token."""
    T, n = z.shape[0], taps.shape[1]
    out = torch.zeros_like(z) + bias
    for t in range(T):
        for back in range(n):
            if t - back >= 0:
                out[t] = out[t] + taps[:, n - 1 - back] * z[t - back]
    return out


def part_products(u, mats, bias):
    """u [T, C] cut into as many equal parts as ``mats`` [parts, size, size] has matrices (rows = outputs)."""
    parts, size = mats.shape[0], mats.shape[1]
    pieces = [u[:, b * size:(b + 1) * size] @ mats[b].T + bias[b] for b in range(parts)]
    return torch.cat(pieces, dim=1)


def decays(r, lam):
    """Logarithm of the decay of every channel: −8 · r · ln(1 + e^lam)."""
    return -DECAY_FACTOR * r * torch.log1p(torch.exp(lam))


def linear_recurrence(log_d, v):
    """S_t = d_t S_{t−1} + sqrt(1 − d_t²) v_t from S = 0, also at the first token."""
    S = torch.zeros_like(v[0])
    out = []
    for t in range(v.shape[0]):
        d = torch.exp(log_d[t])
        S = d * S + torch.sqrt(1.0 - d * d) * v[t]
        out.append(S)
    return torch.stack(out)


def rglru(a, w, p):
    """Mixer 'rglru'."""
    y = gelu_tanh(a @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(a @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = torch.sigmoid(part_products(u, w[p + "ra"], w[p + "ra.b"]))
    i = torch.sigmoid(part_products(u, w[p + "ri"], w[p + "ri.b"]))
    S = linear_recurrence(decays(r, w[p + "lam"]), i * u)
    return (S * y) @ w[p + "o"].T


def rotate_halves(v, base: float):
    """v [T, heads, dims]: dim i pairs with dim i + dims/2, turned by t · base^(−2i/dims)."""
    T, dims = v.shape[0], v.shape[-1]
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64).to(v.dtype)
    ang = torch.arange(T, dtype=v.dtype)[:, None] * freq[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    lo, hi = v[..., :half], v[..., half:]
    return torch.cat([lo * c - hi * s, hi * c + lo * s], dim=-1)


def causal_softmax(s):
    T = s.shape[-1]
    s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], -math.inf)
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def latent_attention(a, w, p, m, eps):
    """Mixer 'latent_attention'."""
    T = a.shape[0]
    H, d, rd, vd, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (a @ w[p + "q"].T).reshape(T, H, d + rd)
    low = a @ w[p + "dkv"].T
    c = rms_norm(low[:, :rank], w[p + "dkv.norm"], eps)
    k = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, vd)
    s = torch.einsum("ihd,jhd->hij", q[..., :d], k)
    if rd:
        base = m["rot"]["base"]
        s = s + torch.einsum("ihd,jd->hij", rotate_halves(q[..., d:], base), rotate_halves(low[:, None, rank:], base)[:, 0])
    o = torch.einsum("hij,jhv->ihv", causal_softmax(s * m["scale"]), v).reshape(T, H * vd)
    return (o * torch.sigmoid(a @ w[p + "g"].T)) @ w[p + "o"].T


def gelu_gated(a, w, p):
    return (gelu_tanh(a @ w[p + "gate"].T) * (a @ w[p + "up"].T)) @ w[p + "down"].T


def routed_experts(a, w, p, router: dict):
    """``experts`` feed-forwards and ``identity`` places that return the input; a token takes the ``top`` places with
    the largest softmax score + correction, each weighted by its score alone."""
    n, same, top = router["experts"], router.get("identity") or 0, router["top"]
    z = a @ w[p + "router"].T
    e = torch.exp(z - z.max(dim=-1, keepdim=True).values)
    s = e / e.sum(dim=-1, keepdim=True)
    assert s.shape[1] == n + same
    choice = s + w[p + "correction"]
    out = torch.zeros_like(a)
    for t in range(a.shape[0]):
        for j in torch.topk(choice[t], top).indices.tolist():
            if j >= n:
                y = a[t]
            else:
                h = torch.clamp(w[f"{p}e{j}.up"] @ a[t], min=0.0)
                y = w[f"{p}e{j}.down"] @ (h * h)
            out[t] = out[t] + s[t, j] * y
    return out


def layer_runs(cfg: dict) -> list:
    """[(layer, pass whose row is added in front, or None)] in the order the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for p in range(loop["times"]):
        runs += [(i, p if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg: dict, weights: dict, ids, dtype=torch.float64, layers_out: list | None = None):
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer run."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    x = w["embed"][torch.as_tensor(ids, dtype=torch.long)]
    for i, step in layer_runs(cfg):
        layer = cfg["layers"][i]
        p = f"l{i}."
        if step is not None:
            x = x + w["loop.step"][step]
        a = rms_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "rglru":
            y = rglru(a, w, p + "mix.")
        elif layer["type"] == "latent_attention":
            y = latent_attention(a, w, p + "mix.", layer["mixer"], eps)
        else:
            raise ValueError(f"unknown layer type {layer['type']!r}")
        x = x + m * y
        f = layer.get("mlp")
        if f is not None:
            a = rms_norm(x, w[p + "norm2"], eps)
            y = gelu_gated(a, w, p + "mlp.") if f["kind"] == "dense" else routed_experts(a, w, p + "mlp.", f["router"])
            x = x + m * y
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms_norm(x, w["final.norm"], eps) @ w["head"].T) * cfg.get("logit_scale", 1.0)


def generate_greedy(cfg, weights, prompt, n_new: int) -> list:
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(torch.argmax(forward(cfg, weights, ids)[-1])))
    return ids[len(prompt):]
