"""The Luvavik parts and the whole decoder against the plain implementation in ``plain/luvavik_plain.py``.

Each mechanism alone (kernel against its formula: the recurrent block with its ring of inputs and its state, in chunks and
token by token; the latent row with a key part rotated by halves in one page row; gates per element; gelu-gated products on
every kernel that can serve them; the router without renormalised weights, with experts that return their input; squared
relu experts on every kernel; the norm that adds a row first), then small models with random weights under every way of
cutting the work: whole prompts, token-by-token decoding, portions down to two tokens, batches of unequal requests, slots
and pages used again, long decoding, greedy generation through ``Engine.generate``, the trace program and the command line.
Where random weights would hide a fault (one key among many, a tap of the convolution, a state that is lost), the weights
or inputs are made so that it shows.
"""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import pytest
import torch

import luvavik_models as M
import tiny
import traces
from plain import luvavik_plain as P
from spissa_b200 import Engine, SamplingParams

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
PAGE = 64
TOL = {"float32": 2e-5, "bfloat16": 3e-2}      # the largest difference of a logits row, as a share of the largest logit
# a router's choice is a step: where two choice scores lie closer than bfloat16 rounding, a bfloat16 run may take the
# other expert, and the row moves (the 32-bit runs allow none)
CLOSE_CALLS = {"float32": 0.0, "bfloat16": 0.03}


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def worst(got, ref):
    return float((got.double().cpu() - ref.double()).abs().max() / ref.abs().max())


def compare(got, ref, tol, what, allow=0.0):
    """Every row within ``tol`` of the largest logit, but a share ``allow`` of them; no row is broken (NaN)."""
    assert set(got) == set(ref), what
    scale = max(float(v.abs().max()) for v in ref.values())
    errs = sorted((float((row.double() - ref[k].double()).abs().max()) / scale, k) for k, row in got.items())
    assert all(e == e for e, _ in errs), what
    over = [x for x in errs if x[0] > tol]
    assert len(over) <= allow * len(errs), f"{what}: {len(over)} of {len(errs)} rows beyond {tol:.1e}; the worst {errs[-1]}"


def make_step(counts, at, slots):
    """Step arrays of ``counts[b]`` new tokens of sequence b from position ``at[b]`` in slot ``slots[b]`` (0: it sits out)."""
    live = [b for b, n in enumerate(counts) if n > 0]
    ns = [counts[b] for b in live]
    starts = [0]
    for n in ns:
        starts.append(starts[-1] + n)
    return SimpleNamespace(
        seq_start=i32(starts), seq_slot=i32([slots[b] for b in live]), n_seqs=len(live), all_single=all(n == 1 for n in ns),
        max_new=max(ns), token_seq=i32([i for i, n in enumerate(ns) for _ in range(n)]),
        positions=i32([at[b] + t for b, n in zip(live, ns) for t in range(n)]), host=dict(new_counts=list(ns))), live


# ---------------------------------------------------------------------------------------------- the recurrent block alone
def _rec_weights(W, parts, taps, seed, slow):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, k=1.0: k * torch.randn(*s, generator=g)
    size = W // parts
    w = {"conv": r(W, taps, k=0.7), "conv.b": r(W, k=0.3), "ra": r(parts, size, size, k=1.5 / size ** 0.5), "ra.b": r(parts, size),
         "ri": r(parts, size, size, k=1.5 / size ** 0.5), "ri.b": r(parts, size), "y.b": r(W, k=0.5), "x.b": r(W, k=0.5),
         "lam": r(W, k=2.0) + (-6.0 if slow else 0.0)}
    return {k: v.bfloat16().float() for k, v in w.items()}       # exact in either storage type


def _rec_ref(w, y, x):
    """The recurrent block behind its projections: (S ⊙ gelu(y), the convolution's inputs, the states)."""
    d = {k: v.double() for k, v in w.items()}
    z = x.double() + d["x.b"]
    u = P.causal_conv(z, d["conv"], d["conv.b"])
    r = torch.sigmoid(P.part_products(u, d["ra"], d["ra.b"]))
    i = torch.sigmoid(P.part_products(u, d["ri"], d["ri.b"]))
    S = P.linear_recurrence(P.decays(r, d["lam"]), i * u)
    return S * P.gelu_tanh(y.double() + d["y.b"]), z, S


def _rec_kernel_weights(w, dtype):
    flat = lambda k: w[k].reshape(-1).to(DEV).contiguous()
    return dict(yb=flat("y.b"), xb=flat("x.b"), conv=w["conv"].to(DEV).contiguous(), convb=flat("conv.b"), rab=flat("ra.b"), rib=flat("ri.b"),
                decay=(8.0 * torch.log1p(torch.exp(w["lam"].double()))).float().to(DEV),
                ra=w["ra"].to(dtype).to(DEV).contiguous(), ri=w["ri"].to(dtype).to(DEV).contiguous())


REC_CUTS = {
    "whole": [[200, 9, 131]],
    "portions": [[5, 1, 1], [2, 0, 1], [64, 1, 65], [1, 1, 64], [128, 6, 0]],
    "decoding": [[190, 1, 70]] + [[1, 1, 1]] * 8 + [[1, 0, 1], [1, 0, 51]],
    "chunk edges": [[63, 2, 64], [1, 1, 1], [1, 1, 63], [64, 1, 2], [65, 3, 1], [6, 1, 0]],
}


@pytest.mark.parametrize("W,parts,taps", [(64, 4, 4), (96, 1, 3), (50, 5, 1), (130, 2, 2), (256, 2, 4), (120, 5, 6), (320, 4, 5), (33, 1, 4),
                                          (256, 1, 4), (768, 3, 2), (384, 3, 4), (128, 1, 1)])
@pytest.mark.parametrize("kind", ["float32", "bfloat16"])
def test_recurrent_block_in_every_cut(W, parts, taps, kind):
    """Chunks of 64 tokens in parallel and one token at a time agree with the recurrence written out, from zero and from
    what an earlier step left, with decays near one (the first tokens still count at the end) and with strong ones. The
    32-bit kernels stay within 32-bit rounding; on the tensor cores the gates' operands keep sixteen bits."""
    from spissa_b200.csrc import lib as K
    dtype = torch.float32 if kind == "float32" else torch.bfloat16
    lengths, mult = [200, 9, 131], 0.75
    for slow in (True, False):
        w = _rec_weights(W, parts, taps, 7 * W + taps, slow)
        g = torch.Generator().manual_seed(W + taps)
        ys = [torch.randn(n, W, generator=g) for n in lengths]
        xs = [torch.randn(n, W, generator=g) for n in lengths]
        refs = [_rec_ref(w, y, x) for y, x in zip(ys, xs)]
        kw = _rec_kernel_weights(w, dtype)
        for name, cuts in REC_CUTS.items():
            slots, at = [2, 0, 3], [0, 0, 0]
            state = torch.zeros(5, W, device=DEV)
            ring = torch.zeros(5, taps, W, device=DEV) if taps > 1 else None
            state[1] = state[4] = 9.0                            # nobody's slots
            got = [[], [], []]
            for counts in cuts:
                counts = [min(n, lengths[b] - at[b]) for b, n in enumerate(counts)]
                step, live = make_step(counts, at, slots)
                rows = torch.cat([torch.cat([ys[b][at[b]:at[b] + counts[b]], xs[b][at[b]:at[b] + counts[b]]], dim=1) for b in live])
                out = torch.full((rows.shape[0], W), float("nan"), dtype=dtype, device=DEV)
                K.rglru(rows.to(DEV).contiguous(), kw, ring, state, out, step, W, taps, parts, mult)
                o = 0
                for b in live:
                    got[b].append(out[o:o + counts[b]].cpu())
                    o += counts[b]
                    at[b] += counts[b]
            tol = 3e-6 if dtype == torch.float32 else 4.5e-3     # the output's own rounding to bfloat16
            for b in range(3):
                n = at[b]
                assert worst(torch.cat(got[b]), mult * refs[b][0][:n]) <= tol, (name, b, slow)
                # the state is 32-bit in both; gates whose operands are rounded to sixteen bits move it by little
                assert worst(state[slots[b]].cpu(), refs[b][2][n - 1]) <= (3e-6 if dtype == torch.float32 else 5e-5), (name, b, slow)
                if taps > 1:
                    for p in range(max(0, n - taps), n):
                        assert worst(ring[slots[b], p % taps].cpu(), refs[b][1][p]) <= 1e-6
            assert float((state[[1, 4]] - 9.0).abs().max()) == 0.0


def test_a_sequences_recurrence_does_not_depend_on_the_batch():
    """The same sequence alone and among others, in a prompt and decoded: the same numbers, bit for bit."""
    from spissa_b200.csrc import lib as K
    W, parts, taps = 128, 4, 3
    w = _rec_weights(W, parts, taps, 3, True)
    g = torch.Generator().manual_seed(4)
    xs = [torch.randn(n, 2 * W, generator=g).to(DEV) for n in (90, 131, 17, 64, 5, 70, 1, 2, 33, 12)]
    for dtype in (torch.float32, torch.bfloat16):
        kw = _rec_kernel_weights(w, dtype)

        def run(order, n_dec):
            state, ring = torch.zeros(12, W, device=DEV), torch.zeros(12, taps, W, device=DEV)
            at, outs = [0] * len(order), []
            heads = [xs[b].shape[0] - (n_dec if xs[b].shape[0] > n_dec else 0) for b in order]
            for turn in range(1 + n_dec):
                counts = heads if turn == 0 else [1 if xs[b].shape[0] > n_dec else 0 for b in order]
                if not any(counts):
                    continue
                step, live = make_step(counts, at, list(range(1, len(order) + 1)))
                rows = torch.cat([xs[order[i]][at[i]:at[i] + counts[i]] for i in live]).contiguous()
                out = torch.empty(rows.shape[0], W, dtype=dtype, device=DEV)
                K.rglru(rows, kw, ring, state, out, step, W, taps, parts)
                o = 0
                for i in live:
                    if order[i] == 1:
                        outs.append(out[o:o + counts[i]].clone())
                    o += counts[i]
                    at[i] += counts[i]
            return torch.cat(outs), state[order.index(1) + 1]
        alone, s_alone = run([1], 4)
        among, s_among = run([0, 2, 1, 3, 4, 5, 6, 7, 8, 9], 4)
        assert torch.equal(alone, among) and torch.equal(s_alone, s_among)


# ---------------------------------------------------------------------------------------------- the latent row, the gate
@pytest.mark.parametrize("H,d,rd,rank,dtype", [(3, 8, 4, 20, torch.float32), (2, 16, 16, 112, torch.bfloat16), (1, 5, 2, 7, torch.float32),
                                               (4, 24, 0, 40, torch.float32), (2, 12, 6, 33, torch.bfloat16)])
def test_latent_row_with_a_key_part_rotated_by_halves(H, d, rd, rank, dtype):
    from spissa_b200.csrc import lib as K
    from spissa_b200.parts.rope import rotary_inv_freq
    g = torch.Generator().manual_seed(H * d + rank)
    lengths, pages = [70, 9], [[4, 1], [2]]
    base, eps, R = 50.0, 1e-4, rank + rd
    freq = rotary_inv_freq(base, rd, None).to(DEV) if rd else None
    wc = torch.randn(rank, generator=g).to(dtype)
    table = torch.zeros(3, 2, dtype=torch.int32)
    for b, p in enumerate(pages):
        table[b + 1, :len(p)] = torch.tensor(p)
    pool = torch.zeros(6, 1, PAGE, R, dtype=dtype, device=DEV)
    rows = [torch.randn(n, H * (d + rd) + R + 5, generator=g) for n in lengths]
    at = [0, 0]
    q_got = [[], []]
    for counts in ([5, 1], [64, 0], [1, 8]):
        step, live = make_step(counts, at, [1, 2])
        view = SimpleNamespace(page_table=table.to(DEV), page_size=PAGE, token_seq=step.token_seq, positions=step.positions, seq_slot=step.seq_slot)
        proj = torch.cat([rows[b][at[b]:at[b] + counts[b]] for b in live]).to(DEV).contiguous()
        q = torch.empty(proj.shape[0], H * (d + rd), dtype=dtype, device=DEV)
        flat = torch.empty(proj.shape[0], R, dtype=dtype, device=DEV)
        K.latent_rot_store(proj, wc.to(DEV), q, pool, view, None, freq, H, d, rd, rank, 1.0, eps, rows_out=flat, halves=True)
        o = 0
        for b in live:
            q_got[b].append(q[o:o + counts[b]].cpu())
            o += counts[b]
            at[b] += counts[b]
    tol = 2e-6 if dtype == torch.float32 else 4.5e-3
    for b, n in enumerate(lengths):
        x = rows[b].double()
        qq = x[:, :H * (d + rd)].reshape(n, H, d + rd)
        low = x[:, H * (d + rd):H * (d + rd) + R]
        c = P.rms_norm(low[:, :rank], wc.double(), eps)
        want_q, want = qq[..., :d], c
        if rd:
            want_q = torch.cat([want_q, P.rotate_halves(qq[..., d:], base)], dim=-1)
            want = torch.cat([c, P.rotate_halves(low[:, None, rank:], base)[:, 0]], dim=-1)
        assert worst(torch.cat(q_got[b]), want_q.reshape(n, -1)) <= tol
        held = torch.cat([pool[p, 0] for p in pages[b]])[:n].cpu()
        assert worst(held, want) <= tol
    assert torch.equal(flat[0].cpu(), pool[pages[0][69 // PAGE], 0, 69 % PAGE].cpu())       # the same row token by token


@pytest.mark.parametrize("T,C,off,extra,dtype", [(37, 24, 8, 3, torch.float32), (65, 256, 128, 0, torch.bfloat16), (9, 21, 5, 2, torch.bfloat16),
                                                 (130, 64, 12, 4, torch.bfloat16)])
def test_a_gate_for_every_element(T, C, off, extra, dtype):
    from spissa_b200.csrc import lib as K
    g = torch.Generator().manual_seed(T + C)
    x = torch.randn(T, C, generator=g).to(dtype)
    z = 3.0 * torch.randn(T, off + C + extra, generator=g)
    got = x.to(DEV).clone()
    K.gate_elements(got, z.to(DEV)[:, off:off + C], 0.7)
    assert worst(got, x.double() * torch.sigmoid(z[:, off:off + C].double()) * 0.7) <= (1e-6 if dtype == torch.float32 else 4.5e-3)


# ---------------------------------------------------------------------------------------------- feed-forwards and norm
@pytest.mark.parametrize("T", [1, 9, 16, 17, 64, 65, 130, 300, 1100])
@pytest.mark.parametrize("W,F", [(64, 128), (96, 64), (128, 192), (50, 30)])
def test_gelu_gated_products_on_every_kernel(T, W, F):
    """One to a thousand tokens pick the streaming, the small-batch and the tile kernels (split along K or by pairs), sizes
    they refuse the plain product and an element kernel: gelu(gate) · up · factor in all of them."""
    from spissa_b200.csrc import lib as K
    from spissa_b200.parts.linear import GatedLinear
    g = torch.Generator().manual_seed(T + W)
    x, gate, up = torch.randn(T, W, generator=g), torch.randn(F, W, generator=g) * 0.3, torch.randn(F, W, generator=g) * 0.3
    for dtype in (torch.float32, torch.bfloat16):
        xs, gs, us = (t.to(dtype) for t in (x, gate, up))
        lin = GatedLinear(gs.to(DEV), us.to(DEV), K.ACT_GELU, 0.35)
        got = lin(xs.to(DEV), dtype)
        ref = P.gelu_tanh(xs.double() @ gs.double().T) * (xs.double() @ us.double().T) * 0.35
        # (where no kernel applies the activation itself the pre-activations are rounded to bfloat16 as well)
        assert worst(got, ref) <= (3e-6 if dtype == torch.float32 else 4.5e-3 if lin.block else 2e-2)
        K.check_status(torch.device(DEV))


@pytest.mark.parametrize("K_,N", [(8192, 512), (4096, 1024)])
def test_gelu_gated_products_that_split_a_long_row(K_, N):
    from spissa_b200.csrc import lib as K
    from spissa_b200.parts.linear import GatedLinear
    g = torch.Generator().manual_seed(N)
    for T in (5, 40, 100, 200):
        x, gate, up = (torch.randn(*s, generator=g).bfloat16() for s in ((T, K_), (N, K_), (N, K_)))
        got = GatedLinear((gate * 0.02).to(DEV), (up * 0.02).to(DEV), K.ACT_GELU, 1.25)(x.to(DEV), torch.bfloat16)
        gate_, up_ = (gate * 0.02).double(), (up * 0.02).double()
        assert worst(got, P.gelu_tanh(x.double() @ gate_.T) * (x.double() @ up_.T) * 1.25) <= 4.5e-3, T


@pytest.mark.parametrize("E,same,top,factor", [(6, 3, 2, 0.7), (3, 0, 3, 1.0), (12, 1, 5, 1.6), (5, 4, 1, 0.5), (64, 16, 8, 1.0), (2, 5, 6, 0.9)])
def test_router_with_identity_experts_and_squared_relu_experts(E, same, top, factor):
    """The choice reads scores plus correction, the weights the scores alone (their sum stays what it is); places beyond
    the experts return the input times their weight; a token alone gives the same row as in a batch, bit for bit."""
    from spissa_b200.csrc import lib as K
    g = torch.Generator().manual_seed(E + top)
    T, W, F = 77, 24, 12
    x = torch.randn(T, W, generator=g)
    w = {"router": torch.randn(E + same, W, generator=g) * 0.6, "correction": 0.2 * torch.randn(E + same, generator=g)}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = torch.randn(F, W, generator=g) * 0.4, torch.randn(W, F, generator=g) * 0.4
    wd = {k: v.double() for k, v in w.items()}
    ref = factor * P.routed_experts(x.double(), wd, "", dict(experts=E, identity=same, top=top))
    s = torch.softmax(x.double() @ wd["router"].T, dim=1)
    idx = torch.topk(s + wd["correction"], top, dim=1).indices
    ids = torch.empty(T, top, dtype=torch.int32, device=DEV)
    wts = torch.empty(T, top, device=DEV)
    K.moe_select((x @ w["router"].T).to(DEV).contiguous(), w["correction"].to(DEV), ids, wts, top, softmax=True, weight_scale=factor,
                 normalize=False)
    assert torch.equal(ids.cpu().long().sort(dim=1).values, idx.sort(dim=1).values)
    assert worst(wts, factor * s.gather(1, ids.cpu().long())) <= 3e-6
    if same:
        assert bool((idx >= E).any()) and bool((idx < E).any())
    up = torch.stack([w[f"e{e}.up"] for e in range(E)]).to(DEV)
    dn = torch.stack([w[f"e{e}.down"] for e in range(E)]).to(DEV)
    run = lambda xx, ii, ww, y: K.moe_experts(xx, ii, ww, up, dn, y, top, 0.0, 0.0, act=K.ACT_RELU2, identities=same > 0)
    y = torch.full((T, W), 0.25, device=DEV)
    run(x.to(DEV), ids, wts, y)
    assert worst(y - 0.25, ref) <= 1e-5
    y1, y0 = torch.zeros(1, W, device=DEV), torch.zeros(T, W, device=DEV)
    run(x[5:6].to(DEV), ids[5:6].contiguous(), wts[5:6].contiguous(), y1)
    run(x.to(DEV), ids, wts, y0)
    assert torch.equal(y1[0], y0[5])


@pytest.mark.parametrize("T,W,F,E,same,top", [(8, 64, 40, 6, 2, 3), (300, 128, 96, 8, 3, 2), (600, 256, 320, 5, 1, 4), (40, 72, 24, 9, 4, 4),
                                              (700, 128, 256, 4, 0, 1)])
def test_squared_relu_experts_on_the_tensor_cores(T, W, F, E, same, top):
    """A few pairs (``mma.sync`` tiles, narrow ones for a decode step) and many (grouped tcgen05 tiles, expert sizes that
    are no multiple of the tile's width included)."""
    from spissa_b200.csrc import lib as K
    g = torch.Generator().manual_seed(T + F)
    x = torch.randn(T, W, generator=g).bfloat16()
    up = (torch.randn(E, F, W, generator=g) / W ** 0.5).bfloat16()
    dn = (torch.randn(E, W, F, generator=g) / F ** 0.5).bfloat16()
    ids = torch.stack([torch.randperm(E + same, generator=g)[:top] for _ in range(T)]).int()
    wts = torch.rand(T, top, generator=g)
    ref = torch.zeros(T, W, dtype=torch.float64)
    for t in range(T):
        for k in range(top):
            e = int(ids[t, k])
            h = torch.clamp(up[e].double() @ x[t].double(), min=0.0) if e < E else None
            ref[t] += float(wts[t, k]) * (x[t].double() if e >= E else dn[e].double() @ (h * h))
    y = torch.full((T, W), -0.5, device=DEV)
    K.moe_experts(x.to(DEV), ids.to(DEV), wts.to(DEV), up.to(DEV), dn.to(DEV), y, top, 0.0, 0.0, act=K.ACT_RELU2, identities=same > 0)
    K.check_status(torch.device(DEV))
    assert worst(y + 0.5, ref) <= 8e-3


@pytest.mark.parametrize("H", [33, 96, 512, 2048, 4096, 5000])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_norm_that_adds_a_row_to_the_stream_first(H, dtype):
    from spissa_b200.csrc import lib as K
    g = torch.Generator().manual_seed(H)
    x, row, w = torch.randn(19, H, generator=g), torch.randn(H, generator=g), torch.randn(H, generator=g).to(dtype)
    h = x.to(DEV).clone()
    out = torch.empty(19, H, dtype=dtype, device=DEV)
    K.rmsnorm(h, w.to(DEV), out, 1e-3, add=row.to(DEV))
    assert torch.equal(h.cpu(), x + row)
    assert worst(out, P.rms_norm((x + row).double(), w.double(), 1e-3)) <= (2e-6 if dtype == torch.float32 else 4.5e-3)
    y = x.to(DEV).clone()
    K.add_row(y, row.to(DEV))                                   # where the layer's first norm cannot take it
    assert torch.equal(y, h)


# ---------------------------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in M.CONFIGS.items():
        folder = tmp_path_factory.mktemp(f"luvavik_{name}")
        pcfg, w = M.make(cfg, folder, **M.INIT[name])
        out[name] = SimpleNamespace(folder=str(folder), cfg=pcfg, w=w, vocab=cfg["vocab"], memo={})
    return out


def logits_of(m, toks):
    memo = getattr(m, "memo", None)
    key = tuple(toks)
    if memo is not None and key in memo:
        return memo[key]
    out = P.forward(m.cfg, m.w, toks)
    if memo is not None:
        memo[key] = out
    return out


def refs_of(m, reqs):
    return {(rid, i): row for rid, toks in reqs.items() for i, row in enumerate(logits_of(m, toks))}


LENGTHS = {"a": [70, 3, 40, 130, 12, 100], "b": [30, 90, 65, 1, 120, 129], "c": [17, 70, 5, 64, 33, 95], "d": [66, 2, 45, 140, 20, 96],
           "e": [40, 8, 66, 64, 19, 101]}


@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_layer_by_layer_the_residual_stream_follows_plain(models, name):
    """In 32-bit, after every run of every layer; the rows that stand in front of passes included."""
    m = models[name]
    toks = tiny.random_prompt(m.vocab, 75, 9)
    layers = []
    P.forward(m.cfg, m.w, toks, layers_out=layers)
    eng = Engine.from_folder(m.folder, dtype="float32", max_tokens=64 * 2, max_seqs=1)
    seen = []
    for block in eng.model.layers:
        def run(h, step, cache, row=None, real=block.forward):
            real(h, step, cache, row=row)
            seen.append(h.clone())
        block.forward = run
    s = eng.acquire()
    eng.step([(s, toks, [len(toks) - 1])])
    eng.release(s)
    runs = P.layer_runs(m.cfg)
    assert len(seen) == len(layers) == len(runs)
    for i, (got, ref) in enumerate(zip(seen, layers)):
        assert worst(got, ref) <= 1e-5, f"{name}: run {i} (layer {runs[i][0]}, {m.cfg['layers'][runs[i][0]]['type']})"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_every_cut_agrees_with_plain(models, name, dtype, tmp_path):
    m = models[name]
    reqs = {f"r{i}": tiny.random_prompt(m.vocab, n, 31 * i + n) for i, n in enumerate(LENGTHS[name])}
    ref = refs_of(m, reqs)
    decode = {rid: d for rid, d in zip(reqs, [0, 1, 22, 40, 3, 90])}
    cuts = {"whole": traces.whole(reqs), "tail": traces.tail_one_by_one(reqs, 45),
            "ragged": traces.ragged_batches(reqs, 3, decode),
            "ragged_pairs": traces.ragged_batches(dict(reversed(list(reqs.items()))), 2, decode)}
    results = {}
    for cut, steps in cuts.items():
        out = tmp_path / cut
        traces.run_in_process(m.folder, dtype, steps, str(out))          # a cache that holds just this trace: slots and pages come back
        results[cut] = traces.collect(steps, str(out), m.vocab)
        compare(results[cut], ref, TOL[dtype], f"{name}/{dtype}/{cut}", CLOSE_CALLS[dtype])
    for cut in ("tail", "ragged", "ragged_pairs"):
        compare(results[cut], results["whole"], TOL[dtype], f"{name}/{dtype}: {cut} against whole", CLOSE_CALLS[dtype])


@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_portions_of_a_prompt_down_to_two_tokens(models, name):
    m = models[name]
    toks = tiny.random_prompt(m.vocab, 150, 77)
    ref = logits_of(m, toks)
    other = tiny.random_prompt(m.vocab, 80, 78)
    ref_other = logits_of(m, other)
    engine = Engine.from_folder(m.folder, dtype="float32", max_tokens=64 * 6, max_seqs=3)
    for sizes in ([2, 2, 3, 57, 1, 64, 21], [64, 64, 22], [1, 1, 2, 146], [2] * 75):
        s, s2 = engine.acquire(), engine.acquire()
        at, rows, rows2 = 0, [], []
        for n in sizes:
            entries = [(s, toks[at:at + n], list(range(n)))]
            lo2, hi2 = min(at, 80), min(at + n, 80)                      # the second request's portions end earlier
            if hi2 > lo2:
                entries.append((s2, other[lo2:hi2], list(range(hi2 - lo2))))
            got = engine.step(entries).cpu()
            rows.append(got[:n])
            rows2.append(got[n:])
            at += n
        assert worst(torch.cat(rows), ref) <= 2e-5, sizes
        assert worst(torch.cat(rows2), ref_other) <= 2e-5, sizes
        engine.release(s)
        engine.release(s2)
    engine.cache.check()
    assert engine.cache.slots.held_count == 0


def test_slots_and_pages_that_are_used_again_start_clean(models):
    """A slot's states (of every pass) and rings, and its pages, belong to the new sequence from its first token."""
    m = models["a"]
    engine = Engine.from_folder(m.folder, dtype="float32", max_tokens=64 * 3, max_seqs=2)
    for turn in range(3):
        reqs = [tiny.random_prompt(m.vocab, n, 5 * turn + n) for n in ((100, 30), (7, 120), (64, 65))[turn]]
        slots = [engine.acquire() for _ in reqs]
        got = engine.step([(s, r[:-2], [len(r) - 3]) for s, r in zip(slots, reqs)]).cpu()
        for b, r in enumerate(reqs):
            assert worst(got[b], logits_of(m, r[:-2])[-1]) <= 2e-5
        for i in (2, 1):
            got = engine.step([(s, [r[-i]], [0]) for s, r in zip(slots, reqs)]).cpu()
        for b, r in enumerate(reqs):
            assert worst(got[b], logits_of(m, r)[-1]) <= 2e-5
        for s in slots:
            engine.release(s)
        engine.cache.check()


def test_a_step_that_is_rolled_back_leaves_rings_and_states_as_they_were(models):
    m = models["b"]
    engine = Engine.from_folder(m.folder, dtype="float32", max_tokens=64 * 3, max_seqs=2)
    toks = tiny.random_prompt(m.vocab, 40, 3)
    ref = logits_of(m, toks)
    s = engine.acquire()
    engine.step([(s, toks[:30], [])])
    real = engine.model.head.forward

    def fails(x):
        raise RuntimeError("a head that gives up")
    for n in (1, 7):                                            # a decode step, then a portion
        engine.model.head.forward = fails
        with pytest.raises(RuntimeError, match="gives up"):
            engine.step([(s, [5] * n, [0])])
        engine.model.head.forward = real
    rows = torch.cat([engine.step([(s, [t], [0])]).cpu() for t in toks[30:]])
    assert worst(rows, ref[30:]) <= 2e-5
    engine.release(s)


@pytest.mark.parametrize("name", ["a", "d"])
def test_long_decoding(models, name):
    """220 tokens one by one: the ring turns many times, pages fill up and follow one another, states carry on; in a
    replayed graph from the second step of a length bucket on."""
    m = models[name]
    toks = tiny.random_prompt(m.vocab, 230, 3)
    ref = logits_of(m, toks)
    for dtype in ("float32", "bfloat16"):
        engine = Engine.from_folder(m.folder, dtype=dtype, max_tokens=64 * 4, max_seqs=1)
        s = engine.acquire()
        engine.step([(s, toks[:10], [])])
        rows = torch.cat([engine.step([(s, [t], [0])]).cpu() for t in toks[10:]])
        compare({("long", i): r for i, r in enumerate(rows)}, {("long", i): r for i, r in enumerate(ref[10:])}, TOL[dtype], dtype,
                CLOSE_CALLS[dtype])
        engine.release(s)
        engine.cache.check()


def test_the_first_tokens_of_a_sequence(models):
    """Nothing stands before the first token: not the bias of the convolution's input, not what the slot's last sequence
    left in ring, state and rows; the first token enters the recurrence like every other. In a prompt, one by one, and in
    portions shorter than the convolution."""
    for name in ("a", "b", "c", "d"):
        m = models[name]
        engine = Engine.from_folder(m.folder, dtype="float32", max_tokens=64 * 2, max_seqs=1)
        for toks in (tiny.random_prompt(m.vocab, 40, 1), tiny.random_prompt(m.vocab, 8, 2)):
            ref = logits_of(m, toks)
            for sizes in ([len(toks)], [1] * 8, [2, 2, 1, 3], [3, 5]):
                s = engine.acquire()
                at, rows = 0, []
                for n in sizes:
                    rows.append(engine.step([(s, toks[at:at + n], list(range(n)))]).cpu())
                    at += n
                engine.release(s)
                assert worst(torch.cat(rows), ref[:at]) <= 2e-5, (name, sizes)


def _long_case(m, folder, toks, ref, head, max_pages, checks):
    for dtype in ("float32", "bfloat16"):
        eng = Engine.from_folder(folder, dtype=dtype, max_tokens=64 * max_pages, max_seqs=1)
        s = eng.acquire()
        rows = [eng.step([(s, toks[:head], list(range(head)))]).cpu()]
        rows += [eng.step([(s, [t], [0])]).cpu() for t in toks[head:]]
        eng.release(s)
        compare({("p", i): r for i, r in enumerate(torch.cat(rows))}, {("p", i): r for i, r in enumerate(ref)}, TOL[dtype], dtype,
                CLOSE_CALLS[dtype])
        checks(eng, dtype)


def test_sizes_that_the_tensor_core_kernels_take(tmp_path):
    """Parts of 64 and 128 channels, cached rows of 128 and 256 entries, expert sizes of the grouped tiles, gated products
    with the activation in the epilogue: in bfloat16 a prompt of 300 tokens and the decode steps behind it run on the
    tensor-core kernels, in 32-bit on FFMA ones. Both agree with plain."""
    from spissa_b200.csrc import lib as K
    cfg = M.model(128, 180, [M.layer(M.rec(256, 2, 4), M.dense(192)),
                             M.layer(M.lat(4, 32, 32, 32, 96), M.moe(4, 3, 64, identity=2)),
                             M.layer(M.rec(192, 3, 4), M.moe(6, 2, 128, identity=1)),
                             M.layer(M.lat(3, 16, 64, 48, 192), M.dense(128))],
                  loop=(1, 3, 2), mult=0.8, scale=2.5)
    pcfg, w = M.make(cfg, tmp_path, seed=41, std=0.07)
    toks = tiny.random_prompt(180, 330, 8)
    _long_case(None, str(tmp_path), toks, P.forward(pcfg, w, toks), 300, 7,
               lambda eng, dtype: None)
    assert {"rglru", "latent", "attention", "tc_gemm"} <= set(K.loaded_libraries())


@pytest.mark.parametrize("d,rd,vd", [(128, 64, 128), (64, 64, 128), (32, 32, 64)])
def test_whole_prompts_expand_their_own_rows(tmp_path, monkeypatch, d, rd, vd):
    """Latent heads whose key (dim + rot_dim) and value sizes the tcgen05 prompt kernel takes: whole prompts run on it (in
    every pass of the loop, each with rows of its own), a portion behind cached tokens and decode steps over the cached
    rows. All agree with plain."""
    from spissa_b200.csrc import lib as K
    cfg = M.model(128, 150, [M.layer(M.lat(2, d, rd, vd, 96), M.dense(64)), M.layer(M.rec(64, 2, 3))], loop=(0, 2, 2), mult=0.7, scale=1.25)
    pcfg, w = M.make(cfg, tmp_path, seed=43, std=0.07)
    reqs = {"p": tiny.random_prompt(150, 336, 5), "r": tiny.random_prompt(150, 296, 6)}
    ref = {(rid, i): row for rid, toks in reqs.items() for i, row in enumerate(P.forward(pcfg, w, toks))}
    calls = []
    real = K.flash_prefill_tc_rows
    monkeypatch.setattr(K, "flash_prefill_tc_rows", lambda *a, **kw: (calls.append(a[0].shape[0]), real(*a, **kw))[1])
    for dtype in ("float32", "bfloat16"):
        eng = Engine.from_folder(str(tmp_path), dtype=dtype, max_tokens=64 * 14, max_seqs=2)
        calls.clear()
        sp, sr = eng.acquire(), eng.acquire()
        rows = eng.step([(sp, reqs["p"][:330], list(range(330))), (sr, reqs["r"][:290], list(range(290)))]).cpu()
        got = {("p", i): rows[i] for i in range(330)}
        got.update({("r", i): rows[330 + i] for i in range(290)})
        for i in range(6):
            rows = eng.step([(sp, [reqs["p"][330 + i]], [0]), (sr, [reqs["r"][290 + i]], [0])]).cpu()
            got[("p", 330 + i)], got[("r", 290 + i)] = rows[0], rows[1]
        eng.release(sp), eng.release(sr)
        assert calls == ([620] * 2 if dtype == "bfloat16" else []), calls
        compare(got, ref, TOL[dtype], f"{dtype}: two whole prompts")
        calls.clear()
        s = eng.acquire()
        eng.step([(s, reqs["p"][:40], [])])
        rows = eng.step([(s, reqs["p"][40:330], list(range(290)))]).cpu()
        eng.release(s)
        assert calls == []
        compare({("p", 40 + i): rows[i] for i in range(290)}, {k: v for k, v in ref.items() if k[0] == "p" and 40 <= k[1] < 330},
                TOL[dtype], f"{dtype}: a portion behind cached tokens")


# ---------------------------------------------------------------------------------------------- one token that matters
def _plain_base(T, seed):
    return [t if t != M.NEEDLE else M.NEEDLE + 1 for t in tiny.random_prompt(64, T, seed)]


@pytest.mark.parametrize("heads,dim,rot_dim,vdim,rank", [(2, 8, 4, 6, 20), (3, 16, 16, 16, 112), (2, 128, 64, 128, 64), (1, 6, 2, 5, 9)])
def test_a_far_key_among_hundreds(tmp_path, heads, dim, rot_dim, vdim, rank):
    """One row decides, at the start, at page borders and far from both, for the last tokens of a prompt, for a portion
    behind cached tokens and for a decoded token."""
    cfg, patch = M.rows_needle_model(heads, dim, rot_dim, vdim, rank)
    pcfg, w = M.make(cfg, tmp_path, seed=22, std=0.05, patch=patch)
    T = 700
    base = _plain_base(T, 5)
    plain_last = P.forward(pcfg, w, base)[-1]
    engines = {dt: Engine.from_folder(str(tmp_path), dtype=dt, max_tokens=64 * 11, max_seqs=1) for dt in ("float32", "bfloat16")}
    for place in (0, 63, 64, 383, 640):
        toks = M.with_needle(base, place)
        ref = P.forward(pcfg, w, toks)
        assert float((ref[-1] - plain_last).abs().max() / ref[-1].abs().max()) > 0.2
        for dt, eng in engines.items():
            s = eng.acquire()
            head = eng.step([(s, toks[:-1], [T - 2])]).cpu()
            tail = eng.step([(s, [toks[-1]], [0])]).cpu()
            eng.release(s)
            s = eng.acquire()
            eng.step([(s, toks[:500], [])])
            part = eng.step([(s, toks[500:], [T - 501])]).cpu()
            eng.release(s)
            assert worst(head[0], ref[-2]) <= TOL[dt] and worst(tail[0], ref[-1]) <= TOL[dt] and worst(part[0], ref[-1]) <= TOL[dt], (place, dt)


@pytest.mark.parametrize("width,blocks,taps", [(24, 2, 3), (64, 1, 4), (50, 5, 2)])
def test_a_state_that_remembers_hundreds_of_tokens_and_taps_that_reach_just_so_far(tmp_path, width, blocks, taps):
    """Slow decays: a token's mark on the state is still large hundreds of tokens later, across steps and chunks. Fast
    decays: only the convolution reaches back, to its last tap and no further."""
    for slow in (True, False):
        folder = tmp_path / str(slow)
        cfg, patch = M.recurrence_needle_model(width, blocks, taps, slow)
        pcfg, w = M.make(cfg, folder, seed=24, std=0.05, patch=patch)
        engines = {dt: Engine.from_folder(str(folder), dtype=dt, max_tokens=64 * 6, max_seqs=1) for dt in ("float32", "bfloat16")}
        T = 300
        base = _plain_base(T, 6)
        plain_last = P.forward(pcfg, w, base)[-1]
        places = (1, 64, 200) if slow else (T - taps, T - taps - 1, T - 1)
        moved = []
        for place in places:
            toks = M.with_needle(base, place)
            ref = P.forward(pcfg, w, toks)
            moved.append(float((ref[-1] - plain_last).abs().max() / ref[-1].abs().max()))
            for dt, eng in engines.items():
                for sizes in ([T], [T - 1, 1], [100, 150, T - 250], [T - taps] + [1] * taps, [T - 2, 2]):
                    s = eng.acquire()
                    at = 0
                    for n in sizes:
                        got = eng.step([(s, toks[at:at + n], [n - 1])]).cpu()
                        at += n
                    eng.release(s)
                    assert worst(got[0], ref[-1]) <= TOL[dt], (slow, place, dt, sizes)
        if slow:
            assert min(moved) > 0.1, moved
        else:
            assert moved[0] > 0.1 and moved[2] > 0.1 and moved[1] < 0.02, moved       # the edge of the taps shows


# ---------------------------------------------------------------------------------------------- generation, the program
@pytest.mark.parametrize("name", ["a", "d"])
def test_greedy_generation_through_the_entry_point(models, name):
    m = models[name]
    prompts = [tiny.random_prompt(m.vocab, n, 7 * n) for n in (1, 9, 70, 30)]
    engine = Engine.from_folder(m.folder, dtype="float32", max_tokens=64 * 8, max_seqs=3)     # two batches
    results, metrics = engine.generate(prompts, 12, SamplingParams(), stop_ids=[])
    for p, r in zip(prompts, results):
        ids = list(p)
        for tok in r.tokens:                                   # along the engine's own tokens: the chosen one is the largest
            row = logits_of(m, ids)[-1]
            assert float(row.max() - row[tok]) <= 2e-5 * float(row.abs().max()), f"prompt of {len(p)}"
            ids.append(tok)
        assert len(r.tokens) == 12 and r.finish_reason == "length"
    assert metrics.generated_tokens == 12 * len(prompts)
    engine.cache.check()
    assert engine.cache.slots.held_count == 0
    # bfloat16 and sampling run through the same loop
    engine = Engine.from_folder(m.folder, dtype="bfloat16", max_tokens=64 * 8)
    results, _ = engine.generate(prompts, 6, SamplingParams(temperature=0.8, top_k=20, seed=3), stop_ids=[])
    assert all(len(r.tokens) == 6 and all(0 <= t < m.vocab for t in r.tokens) for r in results)


def test_greedy_generation_in_bfloat16_takes_tokens_whose_logits_are_the_largest(models):
    """The greedy head never writes logits; its choice and the logits path's agree along the same tokens."""
    m = models["b"]
    engine = Engine.from_folder(m.folder, dtype="bfloat16", max_tokens=64 * 8)
    prompts = [tiny.random_prompt(m.vocab, n, n) for n in (20, 45)]
    results, _ = engine.generate(prompts, 10, SamplingParams(), stop_ids=[])
    for p, r in zip(prompts, results):
        s = engine.acquire()
        row = engine.step([(s, p, [len(p) - 1])]).cpu()[0]
        for tok in r.tokens:
            assert float(row.max() - row[tok]) <= 2e-2 * float(row.abs().max())
            row = engine.step([(s, [tok], [0])]).cpu()[0]
        engine.release(s)


def test_trace_program_on_a_model_of_this_design(models, tmp_path):
    m = models["b"]
    reqs = {f"q{i}": tiny.random_prompt(m.vocab, n, n) for i, n in enumerate([40, 3, 90])}
    steps = traces.ragged_batches(reqs, 3, {"q0": 5, "q1": 2, "q2": 30})
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype in ("bfloat16", "float32"):
        out = tmp_path / dtype
        proc = subprocess.run(
            [sys.executable, os.path.join(root, "bin", "trace_run"), "--model", m.folder, "--dtype", dtype,
             "--out", str(out), "--max-tokens", str(traces.tokens_needed(steps))],
            input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
        assert proc.returncode == 0, proc.stderr[-2000:]
        compare(traces.collect(steps, str(out), m.vocab), refs_of(m, reqs), TOL[dtype], "trace program", CLOSE_CALLS[dtype])


def test_command_line_generates_from_a_folder_and_from_a_configuration_with_random_weights(models, tmp_path):
    m = models["c"]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    exe = os.path.join(root, "bin", "spissa-b200")
    prompt = tiny.random_prompt(m.vocab, 12, 4)
    proc = subprocess.run([sys.executable, exe, "generate", m.folder, "--token-ids", ",".join(map(str, prompt)),
                           "--max-new-tokens", "5", "--dtype", "fp32", "--ctx", "128"],
                          capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    line = json.loads(proc.stdout.strip().splitlines()[0])
    assert line["tokens"] == P.generate_greedy(m.cfg, m.w, prompt, 5) and line["finish_reason"] == "length"
    cfg_file = tmp_path / "config.json"
    cfg_file.write_text(json.dumps(M.CONFIGS["a"]))
    proc = subprocess.run([sys.executable, exe, "generate", "--random", str(cfg_file), "--token-ids", "1,2,3",
                           "--token-ids", "9,8,7,6,5", "--max-new-tokens", "4", "--temp", "0.7", "--seed", "2", "--ctx", "128"],
                          capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    lines = [json.loads(x) for x in proc.stdout.strip().splitlines()]
    assert [len(x["tokens"]) for x in lines] == [4, 4]
