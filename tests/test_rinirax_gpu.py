"""Rinirax on the GPU against the plain implementation (`rinirax_plain`): each mechanism's kernels
alone, then the engine whole, decoded token by token, in portions down to two tokens, in mixed
batches with pages and state slots used again, with keys far away, at page borders and at a window's
edges, and through the generation entry point, the command line and the replay program."""

from __future__ import annotations

import subprocess
import sys

import pytest
import torch

import rinirax_configs as rc
import rinirax_plain as plain
from mlx_omnia_b200 import GenerationOptions, load
from mlx_omnia_b200.engine.engine import Engine, EngineArgs
from mlx_omnia_b200.engine.step import StepEntry
from mlx_omnia_b200.engine.trace import poison_free_pages
from mlx_omnia_b200.kernels import ops
from mlx_omnia_b200.parts.attention import DifferentialAttention, LatentAttention
from mlx_omnia_b200.parts.base import KVView, LayerContext, PartSpec, Runtime
from trace_tools import ROOT, Trace, stacked

pytestmark = pytest.mark.gpu
CUDA = torch.device("cuda:0")
F64 = torch.float64
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def rel(a, b) -> float:
    a, b = a.detach().cpu().double(), b.detach().cpu().double()
    return float((a - b).abs().max() / b.abs().max().clamp_min(1e-30))


class Batch:
    """A step's metadata for kernels that are called alone: requests that bring `lens` tokens each
    and held `starts` positions before, in state slots `slots`."""

    def __init__(self, lens, starts=None, slots=None):
        starts = starts or [0] * len(lens)
        self.num_seqs, self.q_lens = len(lens), list(lens)
        cu = [0]
        for n in lens:
            cu.append(cu[-1] + n)
        self.num_tokens = cu[-1]
        self.cu_seqlens = torch.tensor(cu, dtype=torch.int32, device=CUDA)
        self.state_slots = torch.tensor(slots or list(range(len(lens))), dtype=torch.int32, device=CUDA)
        self.positions = torch.tensor([s + i for s, n in zip(starts, lens) for i in range(n)], dtype=torch.int32, device=CUDA)
        self.seq_lens = torch.tensor([s + n for s, n in zip(starts, lens)], dtype=torch.int32, device=CUDA)
        self.seq_lens_host = [s + n for s, n in zip(starts, lens)]
        self.max_q_len, self.max_seq_len, self.workspace = max(lens), max(self.seq_lens_host), None
        self.decode_only = all(n == 1 for n in lens)
        self.token_ids = None


# ---- each mechanism alone -------------------------------------------------------------------


class Pages:
    """Shuffled pages, filled with NaN, for a mixer that is stepped on its own: request r's logical page i
    is `order[r][i]`."""

    def __init__(self, mixer, lengths, page, dtype, seed, spare=5):
        self.spec, self.page = mixer.kv_spec(), page
        g = torch.Generator().manual_seed(seed)
        counts = [-(-n // page) for n in lengths]
        shuffled = torch.randperm(sum(counts) + spare, generator=g).tolist()
        self.order, at = [], 0
        for n in counts:
            self.order.append(shuffled[at: at + n])
            at += n
        rows = self.spec.rows
        shape = (len(rows), rows[0][0], page, rows[0][1])
        self.pages = torch.full((sum(counts) + spare, *shape), float("nan"), dtype=dtype, device=CUDA)

    def view(self, starts, lens, writes=True):
        width = max(-(-(s + n) // self.page) for s, n in zip(starts, lens))
        table = torch.full((len(lens), width), -1, dtype=torch.int32)
        slots = []
        for r, (s, n) in enumerate(zip(starts, lens)):
            held = self.order[r][: -(-(s + n) // self.page)]
            table[r, : len(held)] = torch.tensor(held, dtype=torch.int32)
            slots += [self.order[r][t // self.page] * self.page + t % self.page for t in range(s, s + n)]
        return KVView(self.pages, table.to(CUDA), torch.tensor(slots, dtype=torch.int64, device=CUDA), self.page,
                      self.spec.window, writes, self.spec)


def loaded(mixer, weights, dtype):
    """`mixer` with `weights` (checkpoint names without a prefix), kept as the loader keeps them."""
    specs = mixer.tensors()
    assert set(specs) == set(weights)
    mixer.load({k: weights[k].to(torch.float32 if specs[k].kind == "vector" else DTYPES[dtype]).to(CUDA) for k in specs},
               Runtime(DTYPES[dtype], CUDA))
    return mixer


def draw(shapes, seed, gains=None):
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes.items():
        gain = (gains or {}).get(name, 1.0)
        std = gain * shape[-1] ** -0.5 if len(shape) == 2 else gain
        out[name] = (torch.randn(*shape, generator=g) * std).to(torch.bfloat16).float()
    return out


CUTS = [[0, 30, 32, 33, 90, 131] + list(range(132, 139)), [0, 1, 2, 4, 20, 47] + list(range(48, 55))]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,K,rot,page", [(4, 2, 32, 64, 3, 32, 16), (6, 2, 16, 40, 4, 8, 4), (3, 3, 5, 7, 5, 4, 8),
                                                  (4, 1, 64, 128, 4, 64, 16), (2, 2, 48, 96, 1, 48, 16), (1, 1, 9, 20, 2, 0, 4),
                                                  (20, 1, 8, 16, 2, 8, 16), (1, 1, 130, 40, 2, 64, 8)])
def test_differential_attention_over_portions_slots_and_pages(dtype, H, G, dk, dv, K, rot, page):
    """Two requests in portions of 1 to 57 tokens (shorter than the convolution's reach among them), then
    single tokens, from state slots that others used before and shuffled pages filled with NaN; then a
    second mixer with queries and a lambda of its own reads the first one's cache. Two far inputs, one at a
    page's last place, are made loud, so that losing their keys would show."""
    D, eps, scale = 56, 1e-5, 0.9 * dk ** -0.5
    cfg = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": scale, "conv": K, "rot": {"dims": rot, "base": 400.0}}
    position = PartSpec("rotary", {"dims": rot, "theta": 400.0, "pairing": "interleaved"}) if rot else None
    mixers, weights = [], []
    for reads, diff in ((False, 0.3), (True, 0.55)):
        mixer = DifferentialAttention(D, H, G, dk, dv, scale, diff, K, eps, position, own_kv=not reads)
        gains = {"q": 2.5, "k": 2.5} | {n + ".b": 0.3 for n in "qkv"} | {n: 0.6 * dk ** -0.25 for n in ("lq1", "lk1", "lq2", "lk2")}
        weights.append(draw({k: s.shape for k, s in mixer.tensors().items()}, dk + H + reads, gains))
        mixers.append(loaded(mixer, weights[-1], dtype))
    lengths = [cuts[-1] for cuts in CUTS]
    g = torch.Generator().manual_seed(9)
    hs = [torch.randn(n, D, generator=g).to(DTYPES[dtype]) for n in lengths]
    far = [3, 2 * page - 1]  # the latter a page's last place
    for h in hs:
        h[far] *= 4.0
        h[40:] += 0.25 * h[far].sum(0)
    pages = Pages(mixers[0], lengths, page, DTYPES[dtype], 4)
    states = [{"conv": torch.full((5, *m.state_spec()["conv"].shape), 3.0, device=CUDA)} for m in mixers]
    for s in states:
        s["conv"][[3, 1]] = 0.0
    got = [[[], []], [[], []]]
    for i in range(len(CUTS[0]) - 1):
        starts, lens = [c[i] for c in CUTS], [c[i + 1] - c[i] for c in CUTS]
        step = Batch(lens, starts, [3, 1])
        rows = torch.cat([h[s: s + n] for h, s, n in zip(hs, starts, lens)]).to(CUDA)
        for m, mixer in enumerate(mixers):
            out = mixer.forward(rows, LayerContext(step, pages.view(starts, lens, writes=m == 0), states[m], m))
            got[m][0].append(out[: lens[0]])
            got[m][1].append(out[lens[0]:])
    tolerance = 5e-5 if dtype == "float32" else 1e-1
    for r, h in enumerate(hs):
        kept = None
        for m, (w, diff) in enumerate(zip(weights, (0.3, 0.55))):
            want, kept = plain.differential_attention(h.to(F64), w, "", {**cfg, "diff": diff}, eps, kept)
            mine = torch.cat(got[m][r])
            assert rel(mine, want) < tolerance, (r, m)
            if dtype == "bfloat16":  # loud inputs make loud scores, whose rounded queries and keys cost single rows more
                err = (mine.cpu().double() - want).abs().amax(-1) / want.abs().max()
                assert float(err.median()) < 2.5e-2, (r, m)
    for place in far:
        quiet = hs[0].to(F64).clone()
        quiet[place] = 0.0
        lost = plain.differential_attention(quiet, weights[0], "", {**cfg, "diff": 0.3}, eps)[0]
        assert rel(lost[60:], want_of(got[0][0])[60:]) > 1.5 * tolerance
    if K > 1:
        for s in states:
            assert float((s["conv"][[0, 2, 4]] - 3.0).abs().max()) == 0.0  # nobody else's slot was touched
    ops.raise_on_error(CUDA)


def want_of(parts):
    return torch.cat(parts).cpu().double()


@pytest.mark.parametrize("H,G,dk,dv,page", [(4, 1, 64, 128, 16), (2, 2, 32, 64, 16), (3, 3, 48, 96, 16), (4, 2, 24, 20, 8)])
def test_differential_attention_over_a_long_context(H, G, dk, dv, page):
    """A short portion over thousands of keys (few query rows: the key range of a block is cut into parts that are
    merged), then single tokens (split keys) beside another request's portion; one key thousands of positions
    back is made to stand out in one map only, so that either map losing it would show."""
    D, eps, scale, T, K = 40, 1e-6, dk ** -0.5, 2600, 2
    mixer = DifferentialAttention(D, H, G, dk, dv, scale, 0.4, K, eps, PartSpec("rotary", {"dims": 8, "theta": 1e5,
                                                                                        "pairing": "interleaved"}))
    W = draw({k: s.shape for k, s in mixer.tensors().items()}, 3, {n + ".b": 0.1 for n in "qkv"} | {n: 0.5 * dk ** -0.25 for n in
                                                                                                    ("lq1", "lk1", "lq2", "lk2")})
    mixer = loaded(mixer, W, "bfloat16")
    g = torch.Generator().manual_seed(5)
    hs = [torch.randn(T, D, generator=g).to(torch.bfloat16), torch.randn(130, D, generator=g).to(torch.bfloat16)]
    hs[0][77] *= 5.0
    hs[0][2400:] += 0.5 * hs[0][77]
    cuts = [[0, 2100, 2470, 2534, 2536] + list(range(2537, T + 1)), [0, 0, 0, 60, 61] + list(range(62, 62 + T - 2536))]
    pages = Pages(mixer, [T, 130], page, torch.bfloat16, 8)
    state = {"conv": torch.zeros(2, *mixer.state_spec()["conv"].shape, device=CUDA)}
    got = [[], []]
    for i in range(len(cuts[0]) - 1):
        starts, lens = [c[i] for c in cuts], [c[i + 1] - c[i] for c in cuts]
        here = [r for r in (0, 1) if lens[r]]
        step = Batch([lens[r] for r in here], [starts[r] for r in here], here)
        order, pages.order = pages.order, [pages.order[r] for r in here]
        kv = pages.view([starts[r] for r in here], [lens[r] for r in here])
        pages.order = order
        out = mixer.forward(torch.cat([hs[r][starts[r]: starts[r] + lens[r]] for r in here]).to(CUDA), LayerContext(step, kv, state, 0))
        at = 0
        for r in here:
            got[r].append(out[at: at + lens[r]])
            at += lens[r]
    cfg = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": scale, "conv": K, "diff": 0.4, "rot": {"dims": 8, "base": 1e5}}
    for r in (0, 1):
        mine = torch.cat(got[r])
        want = plain.differential_attention(hs[r][: len(mine)].to(F64), W, "", cfg, eps)[0]
        assert rel(mine, want) < 6e-2, r
        if r == 0:
            quiet = hs[0].to(F64).clone()
            quiet[77] = 0.0
            assert rel(plain.differential_attention(quiet, W, "", cfg, eps)[0][2470:], want[2470:]) > 1.2e-1
    ops.raise_on_error(CUDA)


def test_convolution_of_half_split_pairs_and_of_widths_that_are_not_even():
    """The input step alone where no two channels can be taken at once: an odd map width, half-split pairs,
    an amount on cosine and sine; a portion, then single tokens (their state moved on by the second kernel)."""
    H, G, dk, dv, d, K, rot = 2, 1, 7, 5, 16, 3, 6
    C = H * 2 * dk + G * (2 * dk + dv)
    g = torch.Generator().manual_seed(11)
    proj, taps = torch.randn(9, C + 3, generator=g), torch.randn(K, C, generator=g)
    inv = torch.tensor([30.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32, device=CUDA)
    mixer = DifferentialAttention(8, H, G, dk, dv, 1.0, 0.1, K, 1e-5)
    mixer.row = d
    pages = Pages(mixer, [9], 4, torch.float32, 1)
    state, qs = torch.zeros(1, K - 1, C, device=CUDA), []
    for a, b in [(0, 6), (6, 7), (7, 8), (8, 9)]:
        qs.append(ops.conv_heads_prepare(proj[a:b].to(CUDA), 2, None, taps.to(CUDA), state, Batch([b - a], [a]), H, G, 2, dk, dv, d,
                                         inv, True, 1.25, pages.view([a], [b - a])))
    y = plain.causal_conv(proj[:, 2: 2 + C].double(), taps.t())
    pos = torch.arange(9, dtype=F64)[:, None, None] * inv.cpu().double()

    def turned(x):
        u, v = x[..., : rot // 2], x[..., rot // 2: rot]
        c, s = torch.cos(pos) * 1.25, torch.sin(pos) * 1.25
        return torch.cat([u * c - v * s, v * c + u * s, x[..., rot:]], -1)

    q = turned(y[:, : H * 2 * dk].reshape(9, H * 2, dk)).view(9, H, 2, dk)
    want = torch.zeros(9, H, 2, d, dtype=F64)
    want[:, :, 0, :dk], want[:, :, 1, dk: 2 * dk] = q[:, :, 0], q[:, :, 1]
    assert rel(torch.cat(qs).view(9, H, 2, d), want) < 1e-5
    k = turned(y[:, H * 2 * dk: H * 2 * dk + G * 2 * dk].reshape(9, G * 2, dk)).reshape(9, 2 * dk)
    rows = torch.stack([pages.pages[pages.order[0][t // 4], :, 0, t % 4] for t in range(9)]).cpu()
    assert rel(rows[:, 0, : 2 * dk], k) < 1e-5 and rel(rows[:, 1, :dv], y[:, -dv:]) < 1e-5
    assert float(rows[:, 0, 2 * dk:].abs().max()) == 0.0 and float(rows[:, 1, dv:].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,dn,dr,dv,rank,qr,window,scaling,page", [
    (4, 32, 32, 16, 64, 48, 33, (8.0, 256, 16.0, 0.5), 16), (3, 24, 8, 20, 40, 28, 9, (4.0, 64, 8.0, 1.5), 4),
    (5, 12, 6, 10, 20, 12, None, None, 8), (8, 16, 64, 24, 64, 40, 100, (5.0, 1024, 20.0, 2.0), 16),
    (2, 32, 32, 32, 128, 64, 1, None, 16), (6, 64, 64, 64, 256, 96, 257, (40.0, 4096, 32.0, 1.0), 16)])
def test_latent_attention_with_query_latents_and_a_window(dtype, H, dn, dr, dv, rank, qr, window, scaling, page):
    """A prompt of 330 tokens in portions and single tokens over shuffled NaN pages. Behind the window pages
    are handed out as -1, as the cache manager does. The input at the far edge of the last query's window,
    and the one just outside it, are made loud: the first must show, the second must not."""
    D, eps, scale, T = 72, 1e-5, 1.3 * (dn + dr) ** -0.5, 340
    rot = {"dims": dr, "base": 900.0}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    cfg = {"heads": H, "dim": dn, "rot_dim": dr, "vdim": dv, "kv_rank": rank, "scale": scale, "rot": rot}
    if window:
        cfg["mask"] = {"size": window}
    mixer = LatentAttention(D, H, dn, dr, dv, rank, scale, eps, PartSpec("rotary", {"dims": dr, "theta": 900.0, "pairing": "half",
                                                                                   "scaling": scaling}),
                            sink=False, gated=False, window=window, q_rank=qr)
    W = draw({k: s.shape for k, s in mixer.tensors().items()}, rank + H, {"uq": 2.0, "uk": 2.0, "dq.norm": 0.3, "dkv.norm": 0.3})
    W["dq.norm"] += 1.0
    W["dkv.norm"] += 1.0
    mixer = loaded(mixer, W, dtype)
    g = torch.Generator().manual_seed(2)
    h = torch.randn(T, D, generator=g).to(DTYPES[dtype])
    last = T - 1
    inside = last - window + 1 if window else 2
    h[inside] = h[last] * 3.0
    if window and inside:
        h[inside - 1] = h[last] * 3.0
    pages = Pages(mixer, [T], page, DTYPES[dtype], 6)
    got = []
    for a, b in [(0, 129), (129, 131), (131, 200), (200, 330)] + [(t, t + 1) for t in range(330, T)]:
        kv = pages.view([a], [b - a])
        if window:
            dead = max(a - window + 1, 0) // page
            kv.block_table[:, :dead] = -1
        got.append(mixer.forward(h[a:b].to(CUDA), LayerContext(Batch([b - a], [a]), kv, None, 0)))
    want = plain.latent_attention(h.to(F64), W, "", cfg, eps)
    tolerance = 5e-5 if dtype == "float32" else 3e-2
    got = torch.cat(got)
    assert rel(got, want) < tolerance
    if window and window < T and window > 1:
        for place, shows in ((inside, True), (inside - 1, False)):
            other = h.to(F64).clone()
            other[place] = -other[place]
            moved = plain.latent_attention(other, W, "", cfg, eps)
            assert (rel(moved[last], want[last]) > 2 * tolerance) is shows
    ops.raise_on_error(CUDA)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("C,segments", [(48, None), (64, (16, 8)), (30, (3, 2)), (160, (1, 1)), (513, (16, 4)), (40, (5, 8))])
def test_min_gru_over_portions_and_slots(dtype, C, segments):
    """Two requests in portions of 1 to 700 tokens (cut into segments over the warps of a block and the blocks of
    a cluster, more segments than tokens among them) from slots that others used before, then single tokens."""
    g = torch.Generator().manual_seed(C)
    dt = DTYPES[dtype]
    rows = {r: (torch.randn(T, 3 * C + 3, generator=g) * 1.5).to(dt) for r, T in (("a", 796), ("b", 47))}
    zb, ub = torch.randn(C, generator=g) - 2.0, torch.randn(C, generator=g)
    S = torch.full((5, C), 3.0, dtype=torch.float32, device=CUDA)
    S[[3, 1]] = 0.0
    got = {"a": [], "b": []}
    cuts = {"a": [0, 37, 38, 40, 56, 75, 775, 790] + list(range(791, 797)), "b": [0, 1, 2, 3, 19, 20, 21, 41] + list(range(42, 48))}
    for i in range(13):
        a0, a1, b0, b1 = cuts["a"][i], cuts["a"][i + 1], cuts["b"][i], cuts["b"][i + 1]
        step = Batch([a1 - a0, b1 - b0], [a0, b0], [3, 1])
        proj = torch.cat([rows["a"][a0:a1], rows["b"][b0:b1]]).to(CUDA)
        out = ops.mingru(proj, 1, 1 + C, 1 + 2 * C, zb.to(CUDA), ub.to(CUDA), S, step, segments)
        got["a"].append(out[: a1 - a0])
        got["b"].append(out[a1 - a0:])
    for r in rows:
        x = rows[r].to(F64)[:, 1:]
        states = plain.min_gru_states(x[:, :C] + zb.to(F64), x[:, C: 2 * C] + ub.to(F64))
        assert rel(torch.cat(got[r]), states * plain.silu(x[:, 2 * C: 3 * C])) < (2e-5 if dtype == "float32" else 6e-3), r
        assert rel(S[3 if r == "a" else 1], states[-1]) < 2e-5
    assert float((S[[0, 2, 4]] - 3.0).abs().max()) == 0.0
    ops.raise_on_error(CUDA)


def test_a_far_token_shows_through_a_closed_gate():
    """Channel 0's gate stays shut after the first token (its state is carried untouched), channel 1's is open."""
    T, C = 600, 2
    proj = torch.zeros(T, 3 * C)
    proj[:, 0], proj[:, 1], proj[0, 0] = -40.0, 2.0, 40.0
    proj[0, 2:4] = 7.0
    proj[:, 4:] = 1.0
    S, out = torch.zeros(1, C, device=CUDA), []
    for a, b in [(0, 1), (1, 300), (300, 599), (599, 600)]:
        out.append(ops.mingru(proj[a:b].to(CUDA), 0, C, 2 * C, None, None, S, Batch([b - a], [a], [0])))
    assert float(S[0, 0]) == pytest.approx(7.5, rel=1e-5) and float(S[0, 1]) == pytest.approx(0.5, rel=1e-5)
    assert float(torch.cat(out)[-1, 0]) == pytest.approx(7.5 / (1 + 2.718281828 ** -1), rel=1e-5)


@pytest.mark.parametrize("rows", [1, 9, 1300])
@pytest.mark.parametrize("experts,top,count,keep,shift", [(24, 5, 2, 1, 0.0), (12, 3, 4, 2, -3.0), (8, 8, 4, 4, 0.0), (9, 4, 3, 2, -0.8),
                                                          (6, 2, 6, 3, -2.0), (5, 2, 1, 1, 0.5), (256, 8, 8, 4, 0.0), (1, 1, 1, 1, -1.0)])
def test_choice_within_the_best_groups(rows, experts, top, count, keep, shift):
    """The router kernel against the plain choice: the same experts, and weights that are shares of the chosen
    scores; choice scores of either sign, groups of one expert, every group kept."""
    g = torch.Generator().manual_seed(experts + rows)
    hidden = 72
    h, router = torch.randn(rows, hidden, generator=g), torch.randn(experts, hidden, generator=g) * 2.0 * hidden ** -0.5
    correction = torch.randn(experts, generator=g) * 0.3 + shift
    counts = torch.zeros(experts, dtype=torch.int32, device=CUDA)
    choice, weight = ops.moe_route(h.to(CUDA), router.to(CUDA), correction.to(CUDA), experts, top, counts, "sigmoid", count, keep,
                                   True, 1.7)
    r = {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}, "scale": 1.7}
    want, shares = plain.route(h.to(F64) @ router.to(F64).T, correction.to(F64), r)
    got = torch.zeros(rows, experts, dtype=F64).scatter(1, choice.cpu().long(), weight.cpu().double())
    full = torch.zeros(rows, experts, dtype=F64).scatter(1, want, shares)
    same = ((got > 0) == (full > 0)).all(-1)
    assert float((~same).float().mean()) <= 0.002  # two choice scores equal to within rounding, if any
    assert rel(got[same], full[same]) < 1e-5
    assert torch.equal(counts.cpu(), torch.bincount(choice.cpu().flatten().long(), minlength=experts).int())
    if keep < count and experts > count:
        narrow = plain.route(h.to(F64) @ router.to(F64).T, correction.to(F64), {**r, "groups": {"count": 1, "keep": 1}})[0]
        assert rows < 9 or not torch.equal(narrow.sort(-1).values, want.sort(-1).values)  # the groups are not a detail
    ops.raise_on_error(CUDA)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,hidden,inner", [(1, 64, 40), (16, 96, 56), (50, 72, 24), (3, 100, 36)])
def test_xielu_in_and_behind_the_product(dtype, rows, hidden, inner):
    g = torch.Generator().manual_seed(rows + hidden)
    dt = DTYPES[dtype]
    h, up = torch.randn(rows, hidden, generator=g).to(dt), (torch.randn(inner, hidden, generator=g) * 3 * hidden ** -0.5).to(dt)
    p, q = torch.tensor(0.4, dtype=F64), torch.tensor(-0.9, dtype=F64)
    rise, fall = torch.nn.functional.softplus(torch.stack([p, q])).tolist()
    got = ops.linear_act(h.to(CUDA), up.to(CUDA), "xielu", (rise, 0.5 + fall))
    want = plain.xielu(h.to(F64) @ up.to(F64).T, p, q)
    assert rel(got, want) < (1e-5 if dtype == "float32" else 1.5e-2)
    small = torch.tensor([[-1e-4, 1e-4, -3e-3, 0.0]], device=CUDA)
    assert rel(ops.activation(small, "xielu", (rise, 0.5 + fall)), plain.xielu(small.cpu().to(F64), p, q)) < 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,hidden", [(1, 96), (37, 100), (5, 2048), (3, 5), (300, 1000)])
def test_layer_norm_and_the_end_of_a_parallel_block(dtype, rows, hidden):
    """Four layers' ends in a row: each adds its branches (one, two, or a branch and experts' rows), averages the
    results so far and norms; rows with a mean far from zero, so that taking the mean off matters."""
    g = torch.Generator().manual_seed(rows + hidden)
    dt, eps = DTYPES[dtype], 1e-5
    W = {"n": 1.0 + 0.1 * torch.randn(hidden, generator=g), "n.b": 0.2 * torch.randn(hidden, generator=g)}
    x0 = torch.randn(rows, hidden, generator=g) + 30.0
    w, b = W["n"].to(CUDA), W["n.b"].to(CUDA)
    tol = 2e-5 if dtype == "float32" else 8e-3
    assert rel(ops.layernorm(x0.to(CUDA), w, b, eps, dt), plain.layer_norm(x0.double(), W, "n", eps)) < tol
    step = Batch([rows])
    x, want_x, history = x0.to(CUDA), x0.double(), [x0.double()]
    for layer in range(4):
        branch = torch.randn(rows, hidden, generator=g).to(dt)
        r = want_x + branch.double()
        second = None
        if layer == 1:
            second = torch.randn(rows, hidden, generator=g).to(dt)
            r = r + second.double()
            second = second.to(CUDA)
        elif layer == 2:
            top = 3
            outs = torch.randn(rows * top, hidden, generator=g).to(dt)
            place = torch.randperm(rows * top, generator=g).to(torch.int32)
            weight = torch.rand(rows, top, generator=g)
            r = r + (outs.double()[place.long()].view(rows, top, hidden) * weight.double()[..., None]).sum(1)
            second = ops.ExpertRows(outs.to(CUDA), place.to(CUDA), weight.to(CUDA), top)
        coef = torch.randn(layer + 2, generator=g)
        history.append(r)
        want_x = plain.depth_average(history, coef)
        held = ops.depth_history(step, x, 4, layer + 1)
        x, h = ops.depth_step(x, branch.to(CUDA), second, held, coef.to(CUDA), w, b if layer != 3 else None,
                              "rms" if layer == 3 else "layer", eps, keep=layer != 3)
        assert rel(x, want_x) < 1e-5
        want_h = plain.rms(want_x, eps, W["n"]) if layer == 3 else plain.layer_norm(want_x, W, "n", eps)
        assert rel(h, want_h) < tol and h.dtype == dt
    plain_x, none = ops.depth_step(x, branch.to(CUDA), None, None, None, None, None, None, 0.0)
    assert none is None and rel(plain_x, x.cpu().double() + branch.double()) < 1e-6


# ---- the engine -----------------------------------------------------------------------------


def engine_for(name, dtype="float32", page=4, tokens=1024, requests=4, graphs=True, seed=0, raw=None):
    raw = raw or rc.config(name)
    weights = rc.tensors(raw, seed)
    engine = Engine.from_tensors(raw, weights, EngineArgs(dtype=dtype, page_size=page, cache_tokens=tokens,
                                                          max_requests=requests, cuda_graphs=graphs))
    return raw, weights, engine


TOLERANCE = {"float32": 3e-4, "bfloat16": 8e-2}


def every_expert(raw) -> bool:
    """Whether every token uses every expert of every layer (no choice that rounding could turn)."""
    return all(l["mlp"] is None or l["mlp"]["kind"] == "dense" or l["mlp"]["router"]["top"] == l["mlp"]["router"]["experts"] for l in raw["layers"])


def assert_rows(got, want, dtype, what="", tolerance=None, strict=False):
    """Rows of logits against rows of the plain implementation. float32: every row within the tolerance
    (of the largest logit). bfloat16: the median row within a third of it and at most one row in ten
    beyond it: a routed layer's choice between two nearly equal scores can fall the other way than in
    float64, which moves that row by tens of per cent and, through the states and the cache, the rows
    after it by a little; with these configurations' few experts that happens to a few rows in a hundred.
    `strict` (a configuration without such choices): every row within the tolerance in bfloat16 too."""
    tolerance = tolerance or TOLERANCE[dtype]
    got, want = got.detach().cpu().double(), want.detach().cpu().double()
    assert got.shape == want.shape
    err = (got - want).abs().amax(-1) / want.abs().max().clamp_min(1e-30)
    assert not torch.isnan(err).any(), what
    if dtype == "float32" or strict:
        assert float(err.max()) < tolerance, (what, int(err.argmax()), float(err.max()))
    else:
        assert float(err.median()) < tolerance / 3, (what, float(err.median()))
        assert int((err >= tolerance).sum()) <= max(3, len(err) // 10), (what, err.topk(min(5, len(err))))


@pytest.mark.parametrize("name", sorted(rc.CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts(name, dtype):
    raw, weights, engine = engine_for(name, dtype)
    for n in (1, 2, 3, 41, 230):
        ids = rc.prompt(n, raw["vocab"], n)
        request = engine.cache.open("r")
        got = engine.runner.run([StepEntry(request, ids, list(range(n)))])
        engine.cache.close("r")
        assert_rows(got, plain.forward(ids, weights, raw), dtype, n, strict=every_expert(raw))
    ops.raise_on_error(CUDA)


@pytest.mark.parametrize("name,page", [("S", 4), ("T", 16), ("W", 8)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_decoding_and_mixed_batches(tmp_path, name, page, dtype):
    """Six requests over four state slots: prompts read whole, in portions of 2 to 9 tokens and
    token by token, decoded tokens beside portions of other requests, requests that end and whose
    pages and slots the next ones take (free pages are filled with NaN before every step)."""
    raw, weights, engine = engine_for(name, dtype, page=page, tokens=448)
    V = raw["vocab"]
    ids = {r: rc.prompt(n, V, i) for i, (r, n) in enumerate({"a": 170, "b": 33, "c": 2, "d": 58, "e": 60, "f": 17}.items())}
    trace = Trace()
    at = {r: 0 for r in ids}

    def take(r, n):
        out = ids[r][at[r]: at[r] + n]
        at[r] += len(out)
        return out

    trace.step({"a": take("a", 9), "b": take("b", 33)})
    trace.step({"a": take("a", 2), "c": take("c", 1), "d": take("d", 5)}, end=["b"])
    trace.step({"a": take("a", 7), "c": take("c", 1), "d": take("d", 3), "e": take("e", 40)}, end=["c"])
    for _ in range(6):
        trace.step({"a": take("a", 1), "d": take("d", 2), "e": take("e", 1)})
    trace.step({"f": take("f", 17), "a": take("a", 1)}, end=["f"])
    for _ in range(3):
        trace.step({"e": take("e", 1), "a": take("a", 4), "d": take("d", 1)})
    trace.step({"a": take("a", 97)})
    for _ in range(12):
        trace.step({"a": take("a", 1), "d": take("d", 1)})
    trace.step({"a": take("a", 170), "d": take("d", 58), "e": take("e", 60)}, end=["a", "d", "e"])
    got = trace.run_engine(engine, tmp_path / "out", before_step=lambda e, record: poison_free_pages(e))
    assert not engine.cache.requests
    engine.cache.check()
    for r in ids:
        positions, logits = stacked(got[r])
        assert positions == list(range(len(ids[r])))
        assert_rows(logits, plain.forward(ids[r], weights, raw), dtype, r, strict=every_expert(raw))


@pytest.mark.parametrize("name", sorted(rc.CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_equals_decoding_token_by_token(name, dtype):
    """The same prompt whole, and one token a step (captured decode steps, and launched one by one)."""
    for graphs in (True, False):
        raw, weights, engine = engine_for(name, dtype, graphs=graphs)
        ids = rc.prompt(75, raw["vocab"], 77)
        request = engine.cache.open("w")
        whole = engine.runner.run([StepEntry(request, ids, list(range(len(ids))))])
        engine.cache.close("w")
        request = engine.cache.open("t")
        single = torch.cat([engine.runner.run([StepEntry(request, [t], [0])]) for t in ids])
        engine.cache.close("t")
        assert_rows(single, whole, dtype, "token by token against whole", 3e-5 if dtype == "float32" else 6e-2,
                    strict=every_expert(raw))
        assert_rows(single, plain.forward(ids, weights, raw), dtype, strict=every_expert(raw))
    ops.raise_on_error(CUDA)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompts_across_tiles_chunks_and_pages(dtype):
    """700 tokens: portions that start and end inside tiles of 64 keys, decode chunks of
    128 and pages of 16, the last token a repeat of an early one, then 40 tokens decoded beside a short
    request whose pages are the ones nobody held before."""
    raw, weights, engine = engine_for("T", dtype, page=16, tokens=1024)
    ids = rc.prompt(700, raw["vocab"], 5)
    ids[-1] = ids[11]
    other = rc.prompt(50, raw["vocab"], 6)
    a = engine.cache.open("a")
    rows = {}
    at = 0
    for n in (193, 2, 130, 61, 255, 19):
        out = engine.runner.run([StepEntry(a, ids[at: at + n], [n - 1])])
        rows[at + n - 1] = out[0]
        at += n
    b = engine.cache.open("b")
    engine.runner.run([StepEntry(b, other[:10], [])])
    for t in range(at, 700):
        out = engine.runner.run([StepEntry(a, ids[t: t + 1], [0]), StepEntry(b, other[10 + t - at: 11 + t - at], [0])])
        rows[t] = out[0]
        rows[("b", 10 + t - at)] = out[1]
    expect, expect_b = plain.forward(ids, weights, raw), plain.forward(other, weights, raw)
    keys = list(rows)
    assert_rows(torch.stack([rows[key] for key in keys]),
                torch.stack([expect_b[key[1]] if isinstance(key, tuple) else expect[key] for key in keys]), dtype, keys,
                strict=True)
    ops.raise_on_error(CUDA)


def test_the_constants_show_in_the_logits():
    """A constant moved a little: each moves the plain implementation's logits by far more than the engine is
    from it, so the comparisons above see such a fault. In a prompt and in decoding."""
    raw, weights, engine = engine_for("S", "float32")
    ids = rc.prompt(80, raw["vocab"], 8)
    request = engine.cache.open("r")
    got = [engine.runner.run([StepEntry(request, ids[:50], list(range(50)))])]
    got += [engine.runner.run([StepEntry(request, [t], [0])]) for t in ids[50:]]
    expect = plain.forward(ids, weights, raw)
    assert rel(torch.cat(got), expect) < TOLERANCE["float32"]

    def moved(change):
        other = rc.config("S")
        change(other["layers"])
        out = plain.forward(ids, weights, other)
        return min(rel(out[:50], expect[:50]), rel(out[50:], expect[50:]))

    assert moved(lambda l: l[0]["mixer"].update(diff=0.3)) > 1e-3
    assert moved(lambda l: l[3]["mixer"].update(diff=0.5)) > 1e-3
    assert moved(lambda l: l[0]["mixer"].update(scale=0.35)) > 1e-3
    assert moved(lambda l: l[3]["mixer"].update(scale=0.3)) > 1e-3
    assert moved(lambda l: l[0]["mixer"]["rot"].update(dims=6)) > 1e-3
    assert moved(lambda l: l[3]["mixer"]["rot"].update(base=200.0)) > 1e-3
    assert moved(lambda l: l[2]["mixer"].update(scale=0.25)) > 1e-3
    assert moved(lambda l: l[2]["mixer"]["mask"].update(size=10)) > 1e-3
    assert moved(lambda l: l[2]["mixer"]["rot"].update(base=1000.0)) > 1e-3
    assert moved(lambda l: l[2]["mixer"]["rot"]["scaling"].update(factor=3.0)) > 1e-3
    assert moved(lambda l: l[2]["mixer"]["rot"]["scaling"].update(slow=0.5)) > 1e-3
    assert moved(lambda l: l[2]["mixer"]["rot"]["scaling"].update(original=640)) > 1e-3
    assert moved(lambda l: l[0]["mlp"]["router"].update(scale=1.9)) > 1e-3
    assert moved(lambda l: l[0]["mlp"]["router"]["groups"].update(keep=4)) > 1e-3
    assert moved(lambda l: l[4]["mlp"]["router"].update(top=1)) > 1e-3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window,page,rank,rot", [(9, 4, 40, 8), (16, 16, 64, 32), (33, 8, 64, 32), (1, 4, 40, 8)])
def test_a_token_enters_and_leaves_a_window(dtype, window, page, rank, rot):
    """One layer of windowed attention alone: a token changed at position p moves the logits of p to
    p + window - 1 and, to the last bit, of no other place, in a prompt, in portions and in decoding, with
    pages given back behind the window."""
    raw = {"architecture": "Rinirax", "vocab": 97, "width": 64, "norm": {"eps": 1e-6},
           "layers": [{"type": "latent_attention", "mlp": None,
                       "mixer": {"heads": 2, "dim": 16, "rot_dim": rot, "vdim": 16, "kv_rank": rank, "q_rank": 24, "scale": 0.2,
                                 "mask": {"size": window}, "rot": {"base": 100.0, "dims": rot}}}]}
    weights = rc.tensors(raw, 1)
    engine = Engine.from_tensors(raw, weights, EngineArgs(dtype=dtype, page_size=page, cache_tokens=256, max_requests=2))
    ids, p = rc.prompt(90, 97, 3), 41

    def run(tokens, cuts):
        request, out, at = engine.cache.open("r"), [], 0
        for n in cuts:
            poison_free_pages(engine)
            out.append(engine.runner.run([StepEntry(request, tokens[at: at + n], list(range(n)))]).cpu())
            at += n
        engine.cache.close("r")
        return torch.cat(out)

    other = list(ids)
    other[p] = (other[p] + 1) % 97
    for cuts in ([90], [20, 2, 19, 9, 40], [42] + [1] * 48):
        base, moved = run(ids, cuts), run(other, cuts)
        assert_rows(base, plain.forward(ids, weights, raw), dtype, strict=True)
        changed = ((base - moved).abs().amax(-1) > 0).nonzero().flatten().tolist()
        assert changed == list(range(p, min(p + window, 90)))
    ops.raise_on_error(CUDA)


def test_layers_without_pages_and_a_model_of_one_recurrence():
    """Nothing in the paged cache at all: states only, through the same cache manager and captured steps."""
    raw = {"architecture": "Rinirax", "vocab": 64, "width": 40, "norm": {"eps": 1e-5},
           "layers": [{"type": "mingru", "mixer": {"width": 24}, "mlp": None}, {"type": "mingru", "mixer": {"width": 64},
                                                                               "mlp": {"kind": "dense", "ff": 16}}]}
    weights = rc.tensors(raw, 2)
    engine = Engine.from_tensors(raw, weights, EngineArgs(dtype="float32", page_size=4, cache_tokens=64, max_requests=2))
    ids = rc.prompt(60, 64, 4)
    request = engine.cache.open("r")
    got = [engine.runner.run([StepEntry(request, ids[:23], list(range(23)))])]
    got += [engine.runner.run([StepEntry(request, [t], [0])]) for t in ids[23:]]
    assert_rows(torch.cat(got), plain.forward(ids, weights, raw), "float32")


def test_greedy_generation_long_decoding_and_the_scheduler(tmp_path):
    """Through `load(...).generate`: the scheduler admits, batches and chunks; greedy ids are the plain
    implementation's best, 200 tokens past a two-token prompt included (the states are carried through
    all of them)."""
    raw = rc.config("S")
    weights = rc.tensors("S", 3)
    folder = tmp_path / "m"
    rc.write_folder(folder, raw, weights)
    model = load(folder, dtype="float32", page_size=8, cache_tokens=1024, max_requests=4, max_tokens_per_step=16)
    prompts = [rc.prompt(n, raw["vocab"], 20 + n) for n in (2, 5, 23, 40, 9, 31)]
    counts = [200, 12, 12, 12, 12, 12]
    got = [model.generate([prompts[0]], GenerationOptions(max_tokens=200, stop=()))[0]]
    got += model.generate(prompts[1:], GenerationOptions(max_tokens=12, stop=()))
    for prompt, ids, count in zip(prompts, got, counts):
        assert len(ids) == count
        logits = plain.forward(prompt + ids, weights, raw)[len(prompt) - 1: -1]
        best = logits.max(dim=-1).values
        chosen = logits[torch.arange(count), torch.tensor(ids)]
        assert float((best - chosen).max()) <= 1e-3 * float(logits.abs().max())
    assert not model.engine.cache.requests
    done = subprocess.run([sys.executable, str(ROOT / "bin" / "omnia"), "run", "-m", str(folder), "--max-tokens", "5",
                           "--temperature", "0", "--dtype", "float32", *map(str, prompts[1])],
                          capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-3000:]
    assert [int(t) for t in done.stdout.split()[:5]] == got[1][:5]


def test_replay_program_on_a_model_folder(tmp_path):
    """`bin/trace_run` as a user runs it, in bfloat16, on a folder written by the random-weights mode."""
    from safetensors.torch import load_file

    from mlx_omnia_b200.weights.random_init import write_random_model

    raw = rc.config("T")
    folder = write_random_model(tmp_path / "m", raw, seed=4)
    weights = {k: v.float() for k, v in load_file(str(folder / "model.safetensors")).items()}
    ids = rc.prompt(90, raw["vocab"], 1)
    trace = Trace()
    trace.step({"p": ids[:50]}, want="last")
    trace.step({"p": ids[50:52], "q": ids[:7]})
    for t in range(52, 90):
        trace.step({"p": ids[t: t + 1]}, end=["p"] if t == 89 else ["q"] if t == 52 else [])
    got = trace.run(folder, "bfloat16", tmp_path / "out", vocab=raw["vocab"])
    expect = plain.forward(ids, weights, raw)
    positions, logits = stacked(got["p"])
    assert positions == [49] + list(range(50, 90))
    assert_rows(logits, expect[positions], "bfloat16", strict=True)
