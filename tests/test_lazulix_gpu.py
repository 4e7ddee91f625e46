"""The Lazulix parts and the whole decoder against the plain implementation in ``plain/lazulix_plain.py``.

Each mechanism alone (kernel against its formula: the matrix memory in chunks on the tensor cores, in chunks in 32-bit and
token by token, with its normaliser and running maximum; biases, norms per head and rotation by halves into the cache; the
attention kernels with key and value rows of different sizes; layer norms of a sublayer's output into the stream; the clamped
unit on every kernel that has it), then small models with random weights under every way of cutting the work: whole prompts,
token-by-token decoding, portions down to two tokens, batches of unequal requests, slots and pages used again, long decoding,
greedy generation through ``Engine.generate``, the trace program and the command line. Where random weights would hide a fault
(one key among many, a memory that is lost), the weights or inputs are made so that it shows.
"""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import pytest
import torch

import lazulix_models as M
import tiny
import traces
from plain import lazulix_plain as P
from spissa_b200 import Engine, SamplingParams

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
PAGE = 64
TOL = {"float32": 2e-5, "bfloat16": 4e-2}      # the largest difference of a logits row, as a share of the largest logit
# unit rms behind a memory whose output is a difference of large terms blows rounding up: bfloat16 runs may have a few such rows
FEW = {"float32": 0.0, "bfloat16": 0.02}


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def worst(got, ref):
    return float((got.double().cpu() - ref.double()).abs().max() / ref.abs().max())


def compare(got, ref, dtype, what):
    """Every row within the type's tolerance of the largest logit, but few; no row is broken (NaN)."""
    tol = TOL[dtype]
    assert set(got) == set(ref), what
    scale = max(float(v.abs().max()) for v in ref.values())
    errs = sorted((float((row.double() - ref[k].double()).abs().max()) / scale, k) for k, row in got.items())
    assert all(e == e for e, _ in errs), what
    over = [x for x in errs if x[0] > tol]
    assert len(over) <= FEW[dtype] * len(errs), f"{what}: {len(over)} of {len(errs)} rows beyond {tol:.1e}; the worst {errs[-1]}"


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
        seq_len=i32([at[b] + n for b, n in zip(live, ns)]), max_len=max(at[b] + n for b, n in zip(live, ns)),
        positions=i32([at[b] + t for b, n in zip(live, ns) for t in range(n)]), host=dict(new_counts=list(ns))), live


# ---------------------------------------------------------------------------------------------- the matrix memory alone
CUTS = {
    "whole": [[300, 9, 131]],
    "portions": [[5, 1, 1], [2, 0, 1], [64, 1, 65], [1, 1, 64], [200, 6, 0], [28, 0, 0]],
    "decoding": [[280, 1, 70]] + [[1, 1, 1]] * 8 + [[1, 0, 1], [11, 0, 51]],
    "chunk edges": [[63, 2, 64], [1, 1, 1], [1, 1, 63], [64, 1, 2], [65, 3, 1], [106, 1, 0]],
    "chunk edges 2": [[127, 3, 128], [1, 1, 1], [129, 2, 2], [43, 3, 0]],
}


def _memory_case(H, d, vd, cap, seed, kind):
    """Projected rows of three sequences (gates without biases) and what the memory makes of them: unit rms of the outputs,
    weight and gate. ``kind``: "mixed" gates, gates that "keep" hundreds of tokens, or that "jump" between their caps."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, k=1.0: k * torch.randn(*s, generator=g)
    ib, fb = r(H), r(H, k=2.0) + (2.0 if kind == "mixed" else 8.0 if kind == "keep" else 0.0)
    norm = 1.0 + 0.3 * r(H * vd)
    spread = 40.0 if kind == "jump" else 1.5
    cases = []
    for n in (300, 9, 131):
        # keys near the queries, up to the sign of n · q: unit rms blows up what rounding leaves of a difference of large terms
        side = r(n, H, 1).sign()
        q = r(n, H * d)
        k, v, gate = q + 0.5 * r(n, H * d), r(n, H * vd), r(n, H * vd)
        q = (side * (q + 1.5).view(n, H, d)).reshape(n, H * d)
        k = k + 1.5
        q, k, v = (x.bfloat16().float() for x in (q, k, v))             # exact in either form of the products
        gi, gf = r(n, H, k=spread), r(n, H, k=spread)
        i, f = P.capped_gates(torch.cat([gi, gf], dim=1).double(),
                              {"i": torch.eye(2 * H)[:H].double(), "f": torch.eye(2 * H)[H:].double(), "i.b": ib.double(), "f.b": fb.double()}, "", cap)
        o, S, nn, m = P.matrix_memory(q.double().view(n, H, d) * d ** -0.5, k.double().view(n, H, d), v.double().view(n, H, vd), i, f)
        y = P.rms_norm(o, 1e-4).reshape(n, H * vd) * norm.double() * torch.sigmoid(gate.double())
        cases.append((torch.cat([q, k, v, gate, gi, gf], dim=1), y, S, nn, m))
    return dict(ib=ib.to(DEV), fb=fb.to(DEV), norm=norm.to(DEV)), cases


@pytest.mark.parametrize("H,d,vd,cap", [(2, 40, 64, 11.0), (1, 5, 9, 2.0), (3, 24, 8, 5.0), (2, 128, 256, 15.0), (1, 16, 320, 8.0), (2, 200, 40, 10.0),
                                        (4, 64, 128, 6.0), (1, 8, 16, 1.0), (2, 72, 48, 13.0), (2, 7, 6, 3.0)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_matrix_memory_in_every_cut(H, d, vd, cap, dtype):
    from spissa_b200.csrc import lib as K
    lengths = [300, 9, 131]
    ld = 2 * H * (d + vd + 1)
    pad = (-ld) % 4                                                     # as the mixer pads its stacked projection
    for kind in ("mixed", "keep", "jump"):
        w, cases = _memory_case(H, d, vd, cap, 3 * H + d + vd, kind)
        for name, cuts in CUTS.items():
            slots, at, got = [2, 0, 3], [0, 0, 0], [[], [], []]
            state, nm = torch.zeros(5, H, d, vd, device=DEV), torch.zeros(5, H, d + 1, device=DEV)
            state[1] = state[4] = nm[1] = nm[4] = 9.0                   # nobody's slots
            for counts in cuts:
                counts = [min(n, lengths[b] - at[b]) for b, n in enumerate(counts)]
                step, live = make_step(counts, at, slots)
                rows = torch.nn.functional.pad(torch.cat([cases[b][0][at[b]:at[b] + counts[b]] for b in live]), (0, pad)).to(DEV).contiguous()
                out = torch.full((rows.shape[0], H * vd), float("nan"), dtype=dtype, device=DEV)
                K.mlstm(rows, w, state, nm, out, step, H, d, vd, cap, 1e-4)
                o = 0
                for b in live:
                    got[b].append(out[o:o + counts[b]].cpu())
                    o += counts[b]
                    at[b] += counts[b]
            K.check_status(torch.device(DEV))
            for b in range(3):
                n, y = at[b], cases[b][1]
                # bfloat16: the output's own rounding, and 2⁻¹⁷ of the products' operands
                tol = 3e-5 if dtype == torch.float32 else 6e-3
                assert worst(torch.cat(got[b]), y[:n]) <= tol, (kind, name, b)
                if n == lengths[b]:
                    _, _, S, nn, m = cases[b]
                    loose = 1e-5 if dtype == torch.float32 else 1e-4
                    assert worst(state[slots[b]], S) <= loose and worst(nm[slots[b], :, :d], nn) <= loose, (kind, name, b)
                    assert float((nm[slots[b], :, d].cpu().double() - m).abs().max()) <= 1e-5
            assert float((state[[1, 4]] - 9.0).abs().max()) == 0.0 and float((nm[[1, 4]] - 9.0).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_sequences_memory_does_not_depend_on_the_batch(dtype):
    """The same sequence alone and among others, in a prompt and decoded: the same numbers, bit for bit."""
    from spissa_b200.csrc import lib as K
    H, d, vd = 2, 16, 32
    g = torch.Generator().manual_seed(4)
    xs = [torch.randn(n, 2 * H * (d + vd + 1), generator=g).to(DEV) for n in (90, 231, 17, 64, 5, 70)]
    w = dict(ib=torch.zeros(H, device=DEV), fb=torch.full((H,), 4.0, device=DEV), norm=torch.ones(H * vd, device=DEV))

    def run(order):
        state, nm = torch.zeros(8, H, d, vd, device=DEV), torch.zeros(8, H, d + 1, device=DEV)
        at, outs = [0] * len(order), []
        for turn in range(5):
            counts = [xs[b].shape[0] - 4 if turn == 0 else 1 for b in order]
            step, live = make_step(counts, at, list(range(1, len(order) + 1)))
            rows = torch.cat([xs[order[i]][at[i]:at[i] + counts[i]] for i in live]).contiguous()
            out = torch.empty(rows.shape[0], H * vd, dtype=dtype, device=DEV)
            K.mlstm(rows, w, state, nm, out, step, H, d, vd, 10.0, 1e-5)
            o = 0
            for i in live:
                if order[i] == 1:
                    outs.append(out[o:o + counts[i]].clone())
                o += counts[i]
                at[i] += counts[i]
        i = order.index(1) + 1
        return torch.cat(outs), state[i], nm[i]
    for x, y in zip(run([1]), run([0, 2, 1, 3, 4, 5])):
        assert torch.equal(x, y)


# ---------------------------------------------------------------------------------------------- q, k and v into the cache
def _paged(lengths, pages, n_pages, g, d, vd, dtype):
    table = torch.zeros(len(lengths) + 1, max(len(p) for p in pages), dtype=torch.int32)
    for b, p in enumerate(pages):
        table[b + 1, :len(p)] = torch.tensor(p)
    kp = torch.zeros(n_pages, g, PAGE, d, dtype=dtype, device=DEV)
    vp = torch.zeros(n_pages, g, PAGE, vd, dtype=dtype, device=DEV)
    return table.to(DEV), kp, vp


@pytest.mark.parametrize("nh,g,d,vd,rd,bias,norm,halves", [
    (4, 2, 24, 16, 8, True, True, True), (3, 3, 10, 7, 6, True, True, True), (6, 1, 64, 64, 64, True, False, True), (2, 2, 128, 40, 0, False, True, True),
    (5, 1, 9, 11, 4, True, False, True), (4, 4, 12, 12, 12, True, True, False), (2, 0, 32, 8, 16, True, True, True), (3, 1, 160, 96, 40, True, True, True)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_biases_norms_rotation_and_store(nh, g, d, vd, rd, bias, norm, halves, dtype):
    """Every head's bias, RMS norm with its weight and rotation at the token's position, into q and the page rows; without
    key heads only the queries move and nothing is cached."""
    from spissa_b200.csrc import lib as K
    from spissa_b200.parts.rope import rotary_amplitude, rotary_inv_freq
    gen = torch.Generator().manual_seed(nh * d + vd)
    lengths, pages = [130, 9], [[4, 1, 5], [2]]
    C = (nh + g) * d + g * vd
    rot = dict(dims=rd, base=40.0, scaling=dict(factor=3.0, original=50, fast=8.0, slow=1.0)) if rd else None
    sc = dict(rot["scaling"], type="ramp") if rd else None
    freq = rotary_inv_freq(40.0, rd, sc).to(DEV) if rd else None
    b = torch.randn(C, generator=gen).to(dtype) if bias else None
    qw, kw = (torch.randn(d, generator=gen).to(dtype) if norm else None for _ in range(2))
    table, kp, vp = _paged(lengths, pages, 7, max(g, 1), d, vd, dtype)
    xs = [torch.randn(n, C + 4, generator=gen) for n in lengths]
    at, q_got = [0, 0], [[], []]
    for counts in ([100, 0], [1, 5], [29, 1], [0, 3]):
        step, live = make_step(counts, at, [1, 2])
        rows = torch.cat([xs[i][at[i]:at[i] + counts[i]] for i in live]).to(DEV).contiguous()
        meta = SimpleNamespace(page_table=table, page_size=PAGE, seq_slot=step.seq_slot, positions=step.positions, token_seq=step.token_seq)
        q = torch.full((rows.shape[0], nh * d), float("nan"), dtype=dtype, device=DEV)
        K.qkv_norm_rot_store(rows, b.to(DEV) if bias else None, q, kp, vp, meta, freq, nh, g, d, vd, rd,
                             q_weight=qw.to(DEV) if norm else None, k_weight=kw.to(DEV) if norm else None, eps=1e-4,
                             rot_mult=rotary_amplitude(sc), halves=halves)
        o = 0
        for i in live:
            q_got[i].append(q[o:o + counts[i]].cpu())
            o += counts[i]
            at[i] += counts[i]
    tol = 4e-6 if dtype == torch.float32 else 4.5e-3

    def placed(x, w):
        x = x.double()
        if norm:
            x = P.rms_norm(x, 1e-4) * w.double()
        if not rd or halves:
            return P.rotate_halves(x, rot)
        perm = list(range(0, rd, 2)) + list(range(1, rd, 2)) + list(range(rd, d))     # neighbouring pairs: the same, reordered
        back = torch.argsort(torch.tensor(perm))
        return P.rotate_halves(x[..., perm], rot)[..., back]
    for i, n in enumerate(lengths):
        x = xs[i][:, :C].double() + (b.double() if bias else 0.0)
        assert worst(torch.cat(q_got[i]), placed(x[:, :nh * d].view(n, nh, d), qw).reshape(n, -1)) <= tol
        if not g:
            continue
        k_ref, v_ref = placed(x[:, nh * d:(nh + g) * d].view(n, g, d), kw), x[:, (nh + g) * d:].view(n, g, vd)
        k_got = torch.cat([kp[p].transpose(0, 1) for p in pages[i]])[:n]
        v_got = torch.cat([vp[p].transpose(0, 1) for p in pages[i]])[:n]
        assert worst(k_got, k_ref) <= tol and worst(v_got, v_ref) <= tol
    if not g:
        assert float(kp.abs().max()) == 0.0 and float(vp.abs().max()) == 0.0
    assert float(kp[[0, 3, 6]].abs().max()) == 0.0 and float(vp[[0, 3, 6]].abs().max()) == 0.0       # nobody's pages


# ---------------------------------------------------------------------------------------------- attention, rows of two sizes
@pytest.mark.parametrize("nh,g,d,vd", [(4, 2, 88, 40), (6, 1, 64, 128), (3, 3, 24, 16), (20, 2, 40, 8), (2, 1, 128, 64), (8, 8, 72, 104), (2, 1, 8, 128),
                                       (4, 1, 160, 96), (4, 2, 56, 56), (32, 1, 32, 16), (2, 2, 7, 5), (5, 1, 128, 128), (1, 1, 104, 24)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_attention_over_rows_of_two_sizes(nh, g, d, vd, dtype):
    """Prompts short and long, portions behind cached tokens and decode steps, in unequal batches, with a score that stands
    out at a far key and at page borders: every kernel that ``attend_paged`` can choose agrees with the formula."""
    from spissa_b200.csrc import lib as K
    from spissa_b200.parts.attention import attend_paged
    gen = torch.Generator().manual_seed(nh + 3 * d + 7 * vd)
    lengths, pages, scale = [420, 65, 130], [[9, 2, 7, 1, 4, 11, 3], [8, 5], [6, 10, 12]], 1.3 * d ** -0.5
    table, kp, vp = _paged(lengths, pages, 13, g, d, vd, dtype)
    qs = [torch.randn(n, nh, d, generator=gen).to(dtype) for n in lengths]
    ks = [torch.randn(n, g, d, generator=gen).to(dtype) for n in lengths]
    vs = [torch.randn(n, g, vd, generator=gen).to(dtype) for n in lengths]
    for j in (0, 63, 64, 200):                                   # keys that the last queries look for
        ks[0][j] = 3.0 * qs[0][419 - j % 5, :: nh // g]
    refs = [P.causal_mix(q.double(), k.double(), v.double(), scale).reshape(-1, nh * vd) for q, k, v in zip(qs, ks, vs)]
    kp += 5.0                                                    # what lies beyond a sequence's end must not matter
    vp += 5.0
    counters = torch.zeros(4096, dtype=torch.int32, device=DEV)
    at, got = [0, 0, 0], [[], [], []]
    for counts in ([300, 0, 70], [20, 30, 1], [90, 30, 0], [1, 1, 0], [1, 1, 1], [1, 1, 1], [1, 0, 1], [1, 0, 1], [5, 2, 55]):
        counts = [min(n, lengths[b] - at[b]) for b, n in enumerate(counts)]
        step, live = make_step(counts, at, [1, 2, 3])
        for b in live:
            for t in range(at[b], at[b] + counts[b]):
                kp[pages[b][t // PAGE], :, t % PAGE], vp[pages[b][t // PAGE], :, t % PAGE] = ks[b][t].to(DEV), vs[b][t].to(DEV)
        cache = SimpleNamespace(k_pool=kp, v_pool=vp, page_table=table, page_size=PAGE, seq_slot=step.seq_slot, positions=step.positions,
                                token_seq=step.token_seq)
        q = torch.cat([qs[b][at[b]:at[b] + counts[b]] for b in live]).reshape(-1, nh * d).to(DEV).contiguous()
        ctx = attend_paged(q, step, cache, nh, g, d, None, scale, counters=counters, vd=vd)
        o = 0
        for b in live:
            got[b].append(ctx[o:o + counts[b]].cpu())
            o += counts[b]
            at[b] += counts[b]
    K.check_status(torch.device(DEV))
    assert at == lengths and int(counters.abs().max()) == 0
    for b in range(3):
        assert worst(torch.cat(got[b]), refs[b]) <= (3e-6 if dtype == torch.float32 else 1.2e-2), b


@pytest.mark.parametrize("window,sink", [(100, False), (None, True), (70, True)])
def test_attention_of_two_sizes_with_windows_and_sinks(window, sink):
    """The options that other mixers ask of the same kernels."""
    from spissa_b200.parts.attention import attend_paged
    nh, g, d, vd, n = 4, 2, 48, 24, 330
    gen = torch.Generator().manual_seed(5)
    table, kp, vp = _paged([n], [[3, 1, 6, 2, 5, 4]], 7, g, d, vd, torch.bfloat16)
    q, k, v = (torch.randn(n, h, s, generator=gen).bfloat16() for h, s in ((nh, d), (g, d), (g, vd)))
    sk = torch.randn(nh, generator=gen) + 2.0 if sink else None
    for t in range(n):
        kp[[3, 1, 6, 2, 5, 4][t // PAGE], :, t % PAGE], vp[[3, 1, 6, 2, 5, 4][t // PAGE], :, t % PAGE] = k[t].to(DEV), v[t].to(DEV)
    s = torch.einsum("ihd,jhd->hij", q.double(), k.double().repeat_interleave(nh // g, dim=1)) * 0.2
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    s = s.masked_fill((j > i) | ((i - j >= window) if window else torch.zeros(n, n, dtype=torch.bool)), float("-inf"))
    e = torch.exp(s)
    den = e.sum(-1, keepdim=True) + (torch.exp(sk.double())[:, None, None] if sink else 0.0)
    ref = torch.einsum("hij,jhv->ihv", e / den, v.double().repeat_interleave(nh // g, dim=1)).reshape(n, -1)
    for counts in ([329], [60]):
        step, _ = make_step([n - counts[0]] if False else counts, [n - 1 - counts[0]], [1])
        cache = SimpleNamespace(k_pool=kp, v_pool=vp, page_table=table, page_size=PAGE, seq_slot=step.seq_slot, positions=step.positions, token_seq=step.token_seq)
        out = attend_paged(q[n - 1 - counts[0]:n - 1].reshape(-1, nh * d).to(DEV).contiguous(), step, cache, nh, g, d, window, 0.2,
                           sink=sk.to(DEV) if sink else None, vd=vd)
        assert worst(out, ref[n - 1 - counts[0]:n - 1]) <= 1.2e-2
    step, _ = make_step([1], [n - 1], [1])
    cache = SimpleNamespace(k_pool=kp, v_pool=vp, page_table=table, page_size=PAGE, seq_slot=step.seq_slot, positions=step.positions, token_seq=step.token_seq)
    out = attend_paged(q[n - 1:].reshape(1, nh * d).to(DEV).contiguous(), step, cache, nh, g, d, window, 0.2, sink=sk.to(DEV) if sink else None, vd=vd)
    assert worst(out, ref[n - 1:]) <= 1.2e-2


# ---------------------------------------------------------------------------------------------- norms, the clamped unit
@pytest.mark.parametrize("W", [33, 96, 512, 1024, 2048, 2052, 4096, 5000, 9000])
@pytest.mark.parametrize("mode", ["last", "next", "raw"])
def test_layer_norm_of_a_sublayers_output_into_the_stream(W, mode):
    from spissa_b200.csrc import lib as K
    g = torch.Generator().manual_seed(W)
    x, y = torch.randn(19, W, generator=g) + 3.0, torch.randn(19, W, generator=g) * 0.1 - 7.0      # means that are not zero
    w1, w2 = torch.randn(W, generator=g), torch.randn(W, generator=g)
    mult = 0.75
    ref = x.double() + mult * P.layer_norm(y.double(), w1.double(), 1e-3)
    nxt = P.layer_norm(ref, w2.double(), 1e-3)
    for dtype in (torch.float32, torch.bfloat16):
        xd, yd = x.to(DEV).clone(), y.to(DEV).clone()
        out = None if mode == "last" else torch.full((19, W), float("nan"), dtype=dtype, device=DEV)
        K.stream_norm_add(xd, yd, w1.to(DEV), mult, 1e-3, w_next=w2.to(DEV) if mode == "next" else None, out=out, raw=mode == "raw", centered=True)
        assert worst(xd, ref) <= 3e-5 and float(yd.abs().max()) == 0.0
        if out is not None:
            assert worst(out, nxt if mode == "next" else ref) <= (5e-5 if dtype == torch.float32 else 4.5e-3)


@pytest.mark.parametrize("rows", [1, 7, 16, 40, 64, 200, 1100])
@pytest.mark.parametrize("H,I", [(64, 128), (96, 192), (40, 24)])
def test_clamped_unit_on_every_kernel(rows, H, I):
    """Limits that bite on both sides: the activation in the epilogue of each product that has it, and behind a plain one."""
    from spissa_b200.csrc import lib as K
    from spissa_b200.parts.linear import GatedLinear
    g = torch.Generator().manual_seed(rows + I)
    for dtype in (torch.float32, torch.bfloat16):
        gate, up = (torch.randn(I, H, generator=g).to(dtype) * 0.3 for _ in range(2))
        x = torch.randn(rows, H, generator=g).to(dtype)
        gl = GatedLinear(gate.to(DEV), up.to(DEV), K.ACT_CLAMPED, limit=0.6, slope=1.702)
        out = gl(x.to(DEV), dtype)
        w = dict(gate=gate.double(), up=up.double(), down=torch.eye(I, dtype=torch.float64))
        ref = P.clamped_unit(x.double(), w, "", 0.6)
        z = x.double() @ gate.double().T
        assert float((z > 0.6).double().mean()) > 0.1 and float((z < -0.6).double().mean()) > 0.1
        assert worst(out, ref) <= (6e-6 if dtype == torch.float32 else 4.5e-3)
        assert bool(gl.block) == (dtype == torch.bfloat16 and I % 64 == 0)
    K.check_status(torch.device(DEV))


# ---------------------------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in M.CONFIGS.items():
        folder = tmp_path_factory.mktemp(f"lazulix_{name}")
        pcfg, w = M.make(cfg, folder, **M.INIT[name])
        out[name] = SimpleNamespace(folder=str(folder), cfg=pcfg, w=w, vocab=cfg["vocab"], memo={})
    return out


def logits_of(m, toks):
    key = tuple(toks)
    if key not in m.memo:
        m.memo[key] = P.forward(m.cfg, m.w, toks)
    return m.memo[key]


def refs_of(m, reqs):
    return {(rid, i): row for rid, toks in reqs.items() for i, row in enumerate(logits_of(m, toks))}


LENGTHS = {"a": [70, 3, 40, 130, 12, 100], "b": [30, 90, 65, 1, 140, 129], "c": [17, 70, 5, 64, 33, 95], "d": [66, 2, 45, 140, 20, 96],
           "e": [40, 8, 66, 64, 19, 101]}


@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_layer_by_layer_the_residual_stream_follows_plain(models, name):
    m = models[name]
    toks = tiny.random_prompt(m.vocab, 75, 9)
    layers = []
    P.forward(m.cfg, m.w, toks, layers_out=layers)
    eng = Engine.from_folder(m.folder, dtype="float32", max_tokens=64 * 2, max_seqs=1)
    seen = []
    for block in eng.model.layers:
        def run(h, step, cache, real=block.forward):
            real(h, step, cache)
            seen.append(h.clone())
        block.forward = run
    s = eng.acquire()
    eng.step([(s, toks, [len(toks) - 1])])
    eng.release(s)
    assert len(seen) == len(layers)
    for i, (got, ref) in enumerate(zip(seen, layers)):
        assert worst(got, ref) <= 2e-5, f"{name}: layer {i} ({m.cfg['layers'][i]['type']})"


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
        compare(results[cut], ref, dtype, f"{name}/{dtype}/{cut}")
    for cut in ("tail", "ragged", "ragged_pairs"):
        compare(results[cut], results["whole"], dtype, f"{name}/{dtype}: {cut} against whole")


@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_portions_of_a_prompt_down_to_two_tokens(models, name):
    m = models[name]
    toks = tiny.random_prompt(m.vocab, 150, 77)
    other = tiny.random_prompt(m.vocab, 80, 78)
    ref, ref_other = logits_of(m, toks), logits_of(m, other)
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
    """A slot's memory, normaliser and maximum, and its pages, belong to the new sequence from its first token."""
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


def test_a_step_that_is_rolled_back_leaves_the_memories_as_they_were(models):
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
    """220 tokens one by one: pages fill up and follow one another, memories carry on; in a replayed graph from the second
    step of a length bucket on."""
    m = models[name]
    toks = tiny.random_prompt(m.vocab, 230, 3)
    ref = logits_of(m, toks)
    for dtype in ("float32", "bfloat16"):
        engine = Engine.from_folder(m.folder, dtype=dtype, max_tokens=64 * 4, max_seqs=1)
        s = engine.acquire()
        engine.step([(s, toks[:10], [])])
        rows = torch.cat([engine.step([(s, [t], [0])]).cpu() for t in toks[10:]])
        compare({("long", i): r for i, r in enumerate(rows)}, {("long", i): r for i, r in enumerate(ref[10:])}, dtype, "long decoding")
        engine.release(s)
        engine.cache.check()


def test_the_first_tokens_of_a_sequence(models):
    """The memory starts at zero and its maximum at 0, whatever the slot's last sequence left; position 0 is not rotated."""
    for name in M.CONFIGS:
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


def test_sizes_that_the_tensor_core_kernels_take(tmp_path):
    """In bfloat16 a prompt of 300 tokens, a portion behind it and decode steps run on the tensor-core kernels (the memory's
    chunks, attention with rows of two sizes and of one, the clamped unit in the epilogue), in 32-bit on FFMA ones. Both agree
    with plain."""
    from spissa_b200.csrc import lib as K
    cfg = M.model(128, 180, [M.layer("attention_2", M.att(4, 2, 80, 48, rot=40, scaling=(2.0, 128, 8.0, 1.0)), M.dense(192, 1.0)),
                             M.layer("mlstm", M.mem(2, 64, 128), M.dense(128)),
                             M.layer("attention_2", M.att(8, 2, 80, 48, rot=40, scaling=(2.0, 128, 8.0, 1.0), kv_from=0), M.dense(64)),
                             M.layer("attention", M.att(4, 1, 64, 64, rot=64), M.dense(128)),
                             M.layer("mlstm", M.mem(1, 128, 264, 8.0))])
    pcfg, w = M.make(cfg, tmp_path, seed=41, std=0.07)
    toks = tiny.random_prompt(180, 390, 8)
    ref = P.forward(pcfg, w, toks)
    for dtype in ("float32", "bfloat16"):
        eng = Engine.from_folder(str(tmp_path), dtype=dtype, max_tokens=64 * 7, max_seqs=1)
        for sizes in ([300] + [1] * 20 + [70], [40, 280, 70]):
            s = eng.acquire()
            at, rows = 0, []
            for n in sizes:
                rows.append(eng.step([(s, toks[at:at + n], list(range(n)))]).cpu())
                at += n
            eng.release(s)
            compare({("p", i): r for i, r in enumerate(torch.cat(rows))}, {("p", i): r for i, r in enumerate(ref)}, dtype, f"{dtype} {sizes[:2]}")
    assert {"mlstm", "attention", "attention_kv", "flash_tc", "tc_gemm"} <= set(K.loaded_libraries())


# ---------------------------------------------------------------------------------------------- one token that matters
def _plain_base(T, seed):
    return [t if t != M.NEEDLE else M.NEEDLE + 1 for t in tiny.random_prompt(64, T, seed)]


@pytest.mark.parametrize("kind,heads,kv,dim,vdim,shared", [("attention", 2, 1, 16, 8, False), ("attention_2", 3, 3, 24, 24, True),
                                                           ("attention_2", 2, 1, 88, 40, False), ("attention", 4, 2, 64, 64, True), ("attention", 1, 1, 10, 5, False)])
def test_a_far_key_among_hundreds(tmp_path, kind, heads, kv, dim, vdim, shared):
    """One key decides, at the start, at page borders and far from both, for the last tokens of a prompt, for a portion behind
    cached tokens and for a decoded token; also through another layer's keys and values."""
    cfg, patch = M.key_needle_model(kind, heads, kv, dim, vdim, shared)
    pcfg, w = M.make(cfg, tmp_path, seed=22, std=0.05, patch=patch)
    T = 700
    base = _plain_base(T, 5)
    plain_last = P.forward(pcfg, w, base)[-1]
    engines = {dt: Engine.from_folder(str(tmp_path), dtype=dt, max_tokens=64 * 11, max_seqs=1) for dt in ("float32", "bfloat16")}
    for place in (0, 63, 64, 383, 640):
        toks = M.with_needle(base, place)
        ref = P.forward(pcfg, w, toks)
        assert float((ref[-1] - plain_last).abs().max() / ref[-1].abs().max()) > 0.15
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


@pytest.mark.parametrize("heads,dim,vdim", [(2, 8, 12), (2, 40, 72), (1, 5, 7)])
def test_a_memory_that_keeps_hundreds_of_tokens_and_one_that_forgets_at_once(tmp_path, heads, dim, vdim):
    """Open forget gates: a token's mark is still large hundreds of tokens later, across steps and chunks. Closed ones: the
    token before the last leaves none."""
    for slow in (True, False):
        folder = tmp_path / str(slow)
        cfg, patch = M.memory_needle_model(heads, dim, vdim, slow)
        pcfg, w = M.make(cfg, folder, seed=24, std=0.05, patch=patch)
        engines = {dt: Engine.from_folder(str(folder), dtype=dt, max_tokens=64 * 6, max_seqs=1) for dt in ("float32", "bfloat16")}
        T = 300
        base = _plain_base(T, 6)
        plain_last = P.forward(pcfg, w, base)[-1]
        moved = []
        for place in (1, 64, 127, 128, 200) if slow else (T - 5,):
            toks = M.with_needle(base, place)
            ref = P.forward(pcfg, w, toks)
            moved.append(float((ref[-1] - plain_last).abs().max() / ref[-1].abs().max()))
            for dt, eng in engines.items():
                for sizes in ([T], [T - 1, 1], [100, 150, T - 250], [T - 5] + [1] * 5, [T - 2, 2]):
                    s = eng.acquire()
                    at = 0
                    for n in sizes:
                        got = eng.step([(s, toks[at:at + n], [n - 1])]).cpu()
                        at += n
                    eng.release(s)
                    assert worst(got[0], ref[-1]) <= TOL[dt], (slow, place, dt, sizes)
        assert min(moved) > 0.1 if slow else max(moved) < 0.02, (slow, moved)


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
        compare(traces.collect(steps, str(out), m.vocab), refs_of(m, reqs), dtype, "trace program")


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
