"""Gisudra on the GPU against the plain implementation (`gisudra_plain`): each mechanism's kernels
alone, then the engine whole, decoded token by token, in portions down to two tokens, in mixed
batches with pages and state slots used again, with keys far away, at page borders, at a window's
edges and among the kept first tokens, and through the generation entry point, the command line and
the replay program."""

from __future__ import annotations

import subprocess
import sys

import pytest
import torch

import gisudra_configs as gc
import gisudra_plain as plain
from mlx_omnia_b200 import GenerationOptions, load
from mlx_omnia_b200.engine.engine import Engine, EngineArgs
from mlx_omnia_b200.engine.step import StepEntry
from mlx_omnia_b200.engine.trace import poison_free_pages
from mlx_omnia_b200.kernels import ops
from mlx_omnia_b200.parts.attention import LatentAttention, SinkWindowAttention
from mlx_omnia_b200.parts.base import KVView, LayerContext, PartSpec, Runtime
from mlx_omnia_b200.parts.feedforward import GLUMLP, RoutedExperts
from mlx_omnia_b200.parts.recurrent import StateSpace
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


class Pages:
    """Shuffled pages, filled with NaN, for mixers that are stepped on their own: request r's logical page i is
    `order[r][i]`. Rows of equal shapes or not."""

    def __init__(self, spec, lengths, page, dtype, seed, spare=5):
        self.spec, self.page = spec, page
        g = torch.Generator().manual_seed(seed)
        counts = [-(-n // page) for n in lengths]
        shuffled = torch.randperm(sum(counts) + spare, generator=g).tolist()
        self.order, at = [], 0
        for n in counts:
            self.order.append(shuffled[at: at + n])
            at += n
        rows = self.spec.rows
        shape = (len(rows), rows[0][0], page, rows[0][1]) if spec.uniform else (spec.elements_per_position * page,)
        self.pages = torch.full((sum(counts) + spare, *shape), float("nan"), dtype=dtype, device=CUDA)

    def view(self, starts, lens):
        """Pages that no query of this step or a later one can read are handed out as -1."""
        width = max(-(-(s + n) // self.page) for s, n in zip(starts, lens))
        table = torch.full((len(lens), width), -1, dtype=torch.int32)
        slots = []
        for r, (s, n) in enumerate(zip(starts, lens)):
            held = list(self.order[r][: -(-(s + n) // self.page)])
            dead = max(self.spec.dead_below(s), 0) // self.page
            for i in range(-(-self.spec.keep_first // self.page), dead):
                held[i] = -1
            table[r, : len(held)] = torch.tensor(held, dtype=torch.int32)
            slots += [self.order[r][t // self.page] * self.page + t % self.page for t in range(s, s + n)]
        return KVView(self.pages, table.to(CUDA), torch.tensor(slots, dtype=torch.int64, device=CUDA), self.page,
                      self.spec.window, True, self.spec)


def loaded(part, weights, dtype):
    """`part` with `weights` (checkpoint names without a prefix), kept as the loader keeps them."""
    specs = part.tensors()
    assert set(specs) == set(weights)
    part.load({k: weights[k].to(torch.float32 if specs[k].kind == "vector" else DTYPES[dtype]).to(CUDA) for k in specs},
              Runtime(DTYPES[dtype], CUDA))
    return part


def draw(part, seed, gains=None):
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, spec in part.tensors().items():
        gain = (gains or {}).get(name, 1.0)
        std = gain * spec.shape[-1] ** -0.5 if len(spec.shape) == 2 else gain
        out[name] = torch.randn(spec.shape, generator=g) * std
        if name.endswith("norm"):
            out[name] = 1.0 + 0.1 * out[name]
        out[name] = out[name].to(torch.bfloat16).float()
    return out


CUTS = [[0, 30, 32, 33, 90, 131] + list(range(132, 139)), [0, 1, 2, 4, 20, 47] + list(range(48, 55))]


# ---- each mechanism alone -------------------------------------------------------------------


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,dv,N,G,K,groups", [(4, 32, 64, 1, 4, 1), (6, 20, 24, 2, 2, 3), (3, 7, 5, 3, 1, 7), (1, 30, 1, 1, 5, 5),
                                               (8, 64, 128, 2, 4, 4), (2, 64, 64, 1, 4, 2), (5, 6, 13, 1, 9, 1), (2, 128, 32, 2, 3, 1),
                                               (2, 16, 256, 1, 16, 1), (16, 64, 16, 4, 4, 8)])
def test_state_space_over_portions_and_slots(dtype, H, dv, N, G, K, groups):
    """Two requests in portions of 1 to 57 tokens (shorter than the convolution's reach among them), then single
    tokens, from state slots that others used before; slow decays, so that the first tokens still show at the end."""
    D, eps = 56, 1e-5
    mixer = StateSpace(D, H, dv, N, G, K, groups, eps)
    W = draw(mixer, H + N, {"in": 1.5, "conv": 1.0, "conv.b": 0.3, "D": 0.7, "A_log": 0.7})
    W["dt_bias"] = W["dt_bias"] - 3.0
    mixer = loaded(mixer, W, dtype)
    cfg = {"heads": H, "vdim": dv, "state": N, "groups": G, "conv": K, "norm_groups": groups}
    lengths = [cuts[-1] for cuts in CUTS]
    g = torch.Generator().manual_seed(9)
    hs = [torch.randn(n, D, generator=g).to(DTYPES[dtype]) for n in lengths]
    state = {name: torch.full((5, *spec.shape), 3.0, device=CUDA) for name, spec in mixer.state_spec().items()}
    for t in state.values():
        t[[3, 1]] = 0.0
    got = [[], []]
    for i in range(len(CUTS[0]) - 1):
        starts, lens = [c[i] for c in CUTS], [c[i + 1] - c[i] for c in CUTS]
        rows = torch.cat([h[s: s + n] for h, s, n in zip(hs, starts, lens)]).to(CUDA)
        out = mixer.forward(rows, LayerContext(Batch(lens, starts, [3, 1]), None, state, 0))
        got[0].append(out[: lens[0]])
        got[1].append(out[lens[0]:])
    for r, h in enumerate(hs):
        want = plain.mamba2(h.to(F64), W, "", cfg, eps)
        assert rel(torch.cat(got[r]), want) < (5e-5 if dtype == "float32" else 3e-2), r
    for name, t in state.items():
        if name == "S" or K > 1:
            assert float((t[[0, 2, 4]] - 3.0).abs().max()) == 0.0  # nobody else's slot was touched
    ops.raise_on_error(CUDA)


def ssd_rows(T, H, dv, N, G, seed):
    """Projected rows z | x | B | C | dt and small tensors of a state-space mixer with one tap of one."""
    g = torch.Generator().manual_seed(seed)
    C = H * dv + 2 * G * N
    rows = torch.randn(T, H * dv + C + H, generator=g)
    w = ops.SSDWeights(torch.ones(C, 1), torch.zeros(C), torch.full((H,), -2.0), torch.zeros(H), torch.zeros(H), torch.ones(H * dv))
    return rows, w


def ssd_plain(rows, w, H, dv, N, G, groups, eps):
    x64 = rows.to(F64)
    inner = H * dv
    z, xbc, dt = torch.split(x64, [inner, inner + 2 * G * N, H], -1)
    xbc = plain.silu(plain.causal_conv(xbc, w.taps, w.conv_bias))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    T = len(rows)
    y, S = plain.state_space(x.view(T, H, dv), B.view(T, G, N), C.view(T, G, N), plain.softplus(dt + w.dt_bias.to(F64)), w.A_log, w.D)
    return plain.gated_group_norm(y.reshape(T, inner), z, groups, eps, w.norm), S


@pytest.mark.parametrize("H,dv,N,G", [(80, 32, 128, 1), (40, 64, 64, 2), (96, 32, 16, 4), (80, 32, 256, 1), (3, 16, 80, 1), (2, 48, 32, 1),
                                      (1, 16, 192, 1), (80, 64, 48, 80), (6, 32, 112, 3), (90, 32, 32, 9), (2, 16, 16, 1)])
def test_the_chunked_recurrence_across_its_edges(H, dv, N, G):
    """Two requests in portions that end inside, at and just past chunks of 64 and 128 tokens, from slots that others
    used, decays from nearly none to a tenth a token. The plain recurrence on x, B and C rounded as the kernel's
    operands are: the carried state must agree to what sums of two float16 numbers hold, far inside one rounding."""
    g = torch.Generator().manual_seed(N + H)
    inner, C, K, eps = H * dv, H * dv + 2 * G * N, 3, 1e-6
    w = ops.SSDWeights(torch.randn(C, K, generator=g) * 0.6, 0.2 * torch.randn(C, generator=g), torch.randn(H, generator=g) - 2.0,
                       torch.linspace(-5.0, 2.0, H), torch.randn(H, generator=g), torch.ones(inner))
    dev = ops.SSDWeights(*(t.to(CUDA) for t in (w.taps, w.conv_bias, w.dt_bias, w.A_log, w.D, w.norm)))
    cuts = [[0, 1, 65, 193, 194, 450, 577], [0, 128, 130, 131, 259, 323, 330]]
    rows = [torch.randn(c[-1], inner + C + H, generator=g).to(torch.bfloat16) for c in cuts]
    S, conv = torch.full((5, H, N, dv), 3.0, device=CUDA), torch.full((5, K - 1, C), 3.0, device=CUDA)
    S[[3, 1]], conv[[3, 1]] = 0.0, 0.0
    exact = S.clone(), conv.clone()
    got, sequential = [[], []], [[], []]
    for i in range(len(cuts[0]) - 1):
        starts, lens = [c[i] for c in cuts], [c[i + 1] - c[i] for c in cuts]
        step = Batch(lens, starts, [3, 1])
        proj = torch.cat([r[a: a + n] for r, a, n in zip(rows, starts, lens)]).to(CUDA)
        for out, states, chunked in ((got, (S, conv), True), (sequential, exact, False)):
            y = ops.ssd_mixer(proj, 0, H, dv, G, N, dev, H, eps, *states, step, chunked=chunked)
            out[0].append(y[: lens[0]])
            out[1].append(y[lens[0]:])
    for r, slot in ((0, 3), (1, 1)):
        z, xbc, dt = torch.split(rows[r].to(F64), [inner, C, H], -1)
        xbc = plain.silu(plain.causal_conv(xbc, w.taps, w.conv_bias))
        dt = plain.softplus(dt + w.dt_bias.to(F64))
        for values, state, out, tolerances in ((xbc.float().to(torch.float16).to(F64), S, got, (5e-5, 6e-3)),
                                               (xbc, exact[0], sequential, (2e-5, 6e-3))):
            x, B, Cc = torch.split(values, [inner, G * N, G * N], -1)
            T = len(values)
            y, held = plain.state_space(x.view(T, H, dv), B.view(T, G, N), Cc.view(T, G, N), dt, w.A_log, w.D)
            assert rel(state[slot], held) < tolerances[0], r
            want = plain.gated_group_norm(y.reshape(T, inner), z, H, eps, w.norm)
            assert rel(torch.cat(out[r]), want) < tolerances[1], r
    assert float((S[[0, 2, 4]] - 3.0).abs().max()) == 0.0
    ops.raise_on_error(CUDA)


def test_a_state_beyond_sixteen_bits_of_exponent():
    """Inputs so large that the state passes float16's range by far: the chunked kernel scales it on its way into the
    product, so its outputs agree with the token-by-token kernel's."""
    T, H, dv, N, G, eps = 300, 2, 32, 16, 1, 1e-6
    rows, w = ssd_rows(T, H, dv, N, G, 5)
    rows[:, H * dv: -H] = rows[:, H * dv: -H].abs() * 120.0
    rows = rows.to(torch.bfloat16).to(CUDA)
    w = ops.SSDWeights(w.taps, w.conv_bias, w.dt_bias, torch.full((H,), -5.0), w.D, w.norm)
    dev = ops.SSDWeights(*(t.to(CUDA) for t in (w.taps, w.conv_bias, w.dt_bias, w.A_log, w.D, w.norm)))
    out, states = [], []
    for chunked in (True, False):
        S, conv = torch.zeros(1, H, N, dv, device=CUDA), torch.zeros(1, 1, H * dv + 2 * G * N, device=CUDA)
        out.append(torch.cat([ops.ssd_mixer(rows[a:b], 0, H, dv, G, N, dev, 2, eps, S, conv, Batch([b - a], [a], [0]), chunked=chunked)
                              for a, b in ((0, 150), (150, 300))]))
        states.append(S)
    assert float(states[1].abs().max()) > 2e5
    assert rel(states[0], states[1]) < 1e-3 and rel(out[0], out[1]) < 8e-3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_token_shows_through_a_slow_decay(dtype):
    """Head 0 hardly decays and its step sizes close after the first token, so what that token wrote is what every
    later one reads, across portions and single tokens; head 1 forgets at once."""
    T, H, dv, N, G = 700, 2, 64, 64, 1
    rows, w = ssd_rows(T, H, dv, N, G, 3)
    inner, at_b = H * dv, 2 * H * dv
    rows[:, -2], rows[:, -1] = -30.0, 6.0
    rows[0, -2] = 3.0
    rows[:, at_b: at_b + 2 * N] = 1.0  # every token's B and C alike
    w = ops.SSDWeights(w.taps, w.conv_bias, torch.zeros(H), torch.tensor([-6.0, 4.0]), w.D, w.norm)
    rows = rows.to(DTYPES[dtype])
    dev = ops.SSDWeights(*(t.to(CUDA) for t in (w.taps, w.conv_bias, w.dt_bias, w.A_log, w.D, w.norm)))
    S, conv = torch.zeros(1, H, N, dv, device=CUDA), torch.zeros(1, 1, H * dv + 2 * G * N, device=CUDA)
    out = []
    for a, b in [(0, 2), (2, 300), (300, 695)] + [(t, t + 1) for t in range(695, T)]:
        out.append(ops.ssd_mixer(rows[a:b].to(CUDA), 0, H, dv, G, N, dev, 2, 1e-6, S, conv, Batch([b - a], [a], [0])))
    want, held = ssd_plain(rows, w, H, dv, N, G, 2, 1e-6)
    assert rel(torch.cat(out), want) < (2e-5 if dtype == "float32" else 1e-2)
    assert rel(S[0, 0], held[0]) < (1e-5 if dtype == "float32" else 1e-2) and float(held[0].abs().max()) > 0.5
    quiet = rows.clone()
    quiet[0] = 0.0
    assert rel(ssd_plain(quiet, w, H, dv, N, G, 2, 1e-6)[0][650:, :dv], want[650:, :dv]) > 0.5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,size,keep,page", [(4, 2, 64, 64, 25, 7, 16), (6, 2, 16, 24, 11, 5, 4), (3, 3, 5, 7, 1, 2, 8),
                                                      (8, 2, 128, 128, 45, 18, 16), (2, 2, 32, 32, None, 0, 16), (4, 1, 96, 96, 33, 16, 16),
                                                      (4, 4, 64, 64, 3, 0, 4), (20, 1, 8, 8, 17, 1, 16), (5, 1, 64, 96, 50, 32, 16)])
def test_windowed_attention_with_kept_tokens_and_mixed_values(dtype, H, G, dk, dv, size, keep, page):
    """Two layers in one pass, the second mixing the first one's values into its own: two requests in portions and
    single tokens over shuffled NaN pages, pages behind the window given back. The last kept token, the one after
    it, the window's last visible token and the one before it are made loud: the visible ones must show in the
    last query, the others must not."""
    D, eps, lam = 56, 1e-5, 0.375
    cfg = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": 1.2 * dk ** -0.5}
    if size is not None:
        cfg["mask"] = {"size": size, "keep_first": keep}
    mixers, weights = [], []
    for kind in ("source", "mixed"):
        mixer = SinkWindowAttention(D, H, G, dk, dv, cfg["scale"], size, keep, eps, gated=True, value_mix=kind)
        weights.append(draw(mixer, dk + H + len(mixers), {"vmix": 0.0}))
        weights[-1]["vmix"] = torch.tensor(lam)
        mixers.append(loaded(mixer, weights[-1], dtype))
    lengths = [cuts[-1] for cuts in CUTS]
    g = torch.Generator().manual_seed(9)
    hs = [[torch.randn(n, D, generator=g).to(DTYPES[dtype]) for n in lengths] for _ in mixers]
    last = lengths[0] - 1
    places = {}
    if size is not None and size > 1:
        if last - size + 1 > keep + 1:
            places = {last - size + 1: True, last - size: False, keep: False} | ({keep - 1: True} if keep else {})
    for place in places:
        hs[1][0][place] = hs[1][0][last] * 3.0
    pages = [Pages(m.kv_spec(), lengths, page, DTYPES[dtype], 4 + i) for i, m in enumerate(mixers)]
    got = [[[], []], [[], []]]
    for i in range(len(CUTS[0]) - 1):
        starts, lens = [c[i] for c in CUTS], [c[i + 1] - c[i] for c in CUTS]
        step = Batch(lens, starts, [3, 1])
        for m, mixer in enumerate(mixers):
            rows = torch.cat([h[s: s + n] for h, s, n in zip(hs[m], starts, lens)]).to(CUDA)
            out = mixer.forward(rows, LayerContext(step, pages[m].view(starts, lens), None, m))
            got[m][0].append(out[: lens[0]])
            got[m][1].append(out[lens[0]:])
    tolerance = 5e-5 if dtype == "float32" else 3e-2
    for r in (0, 1):
        first = None
        for m, w in enumerate(weights):
            want, own = plain.attention(hs[m][r].to(F64), w, "", cfg, eps, first)
            assert rel(torch.cat(got[m][r]), want) < tolerance, (r, m)
            if m == 1:
                unmixed = plain.attention(hs[m][r].to(F64), w, "", cfg, eps, None)[0]
                assert rel(unmixed, want) > 4 * tolerance
            first = own
    first = plain.attention(hs[0][0].to(F64), weights[0], "", cfg, eps, None)[1]
    want = plain.attention(hs[1][0].to(F64), weights[1], "", cfg, eps, first)[0]
    for place, shows in places.items():
        other = hs[1][0].to(F64).clone()
        other[place] = -other[place]
        moved = plain.attention(other, weights[1], "", cfg, eps, first)[0]
        assert (rel(moved[last], want[last]) > 2 * tolerance) is shows, place
    ops.raise_on_error(CUDA)


def test_mixing_needs_the_layer_it_mixes_from():
    mixer = SinkWindowAttention(16, 2, 1, 8, 8, 1.0, 4, 0, 1e-5, gated=True, value_mix="mixed")
    mixer = loaded(mixer, draw(mixer, 1), "float32")
    with pytest.raises(ops.KernelError, match="first_values"):
        mixer.forward(torch.zeros(2, 16, device=CUDA), LayerContext(Batch([2]), Pages(mixer.kv_spec(), [2], 4, torch.float32, 1).view([0], [2]), None, 0))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,dn,dr,dv,rank,size,page", [(4, 32, 32, 48, 64, 33, 16), (3, 24, 8, 20, 40, 9, 4), (5, 12, 6, 10, 20, 14, 8),
                                                       (8, 64, 64, 128, 512, 100, 16), (2, 32, 32, 33, 128, 1, 16),
                                                       (6, 16, 64, 80, 256, 257, 16), (2, 8, 4, 5, 12, None, 16)])
def test_latent_attention_with_a_gate_on_every_value(dtype, H, dn, dr, dv, rank, size, page):
    """A prompt in portions and single tokens over shuffled NaN pages, pages behind the window given back. The input
    at the far edge of the last query's window, and the one just outside it, are made loud: the first must show,
    the second must not."""
    D, eps, T = 72, 1e-5, 340
    cfg = {"heads": H, "dim": dn, "rot_dim": dr, "vdim": dv, "kv_rank": rank, "scale": 1.3 * (dn + dr) ** -0.5,
           "rot": {"base": 900.0, "dims": dr}}
    if size:
        cfg["mask"] = {"size": size}
    mixer = LatentAttention(D, H, dn, dr, dv, rank, cfg["scale"], eps, PartSpec("rotary", {"dims": dr, "theta": 900.0,
                                                                                         "pairing": "interleaved"}),
                            sink=False, gated="values", window=size)
    W = draw(mixer, rank + H, {"q": 2.0, "uk": 2.0})
    mixer = loaded(mixer, W, dtype)
    g = torch.Generator().manual_seed(2)
    h = torch.randn(T, D, generator=g).to(DTYPES[dtype])
    last = T - 1
    inside = last - size + 1 if size else 2
    h[inside] = h[last] * 3.0
    if size and size > 1:
        h[inside - 1] = h[last] * 3.0
    pages = Pages(mixer.kv_spec(), [T], page, DTYPES[dtype], 6)
    got = []
    for a, b in [(0, 129), (129, 131), (131, 200), (200, 330)] + [(t, t + 1) for t in range(330, T)]:
        got.append(mixer.forward(h[a:b].to(CUDA), LayerContext(Batch([b - a], [a]), pages.view([a], [b - a]), None, 0)))
    want = plain.latent_attention(h.to(F64), W, "", cfg, eps)
    tolerance = 5e-5 if dtype == "float32" else 3e-2
    assert rel(torch.cat(got), want) < tolerance
    if size and size > 1:
        for place, shows in ((inside, True), (inside - 1, False)):
            other = h.to(F64).clone()
            other[place] = -other[place]
            moved = plain.latent_attention(other, W, "", cfg, eps)
            assert (rel(moved[last], want[last]) > 2 * tolerance) is shows
    ops.raise_on_error(CUDA)


@pytest.mark.parametrize("rows", [1, 9, 1300])
@pytest.mark.parametrize("experts,top,hidden", [(24, 5, 72), (12, 12, 64), (9, 1, 50), (256, 8, 128), (1, 1, 40), (31, 3, 33)])
def test_choice_by_logits_and_a_softmax_of_the_chosen(rows, experts, top, hidden):
    """The router kernel against the plain choice, with a bias that matters, and the shared expert's gate from the
    router's last row."""
    g = torch.Generator().manual_seed(experts + rows)
    h, router = torch.randn(rows, hidden, generator=g), torch.randn(experts + 1, hidden, generator=g) * 2.0 * hidden ** -0.5
    bias = torch.randn(experts, generator=g)
    counts = torch.zeros(experts, dtype=torch.int32, device=CUDA)
    gate = torch.empty(rows, device=CUDA)
    choice, weight = ops.moe_route(h.to(CUDA), router.to(CUDA), None, experts, top, counts, "chosen", bias=bias.to(CUDA), shared_gate=gate)
    z = h.to(F64) @ router.to(F64).T
    want, shares = plain.route(z[:, :experts] + bias.to(F64), top)
    got = torch.zeros(rows, experts, dtype=F64).scatter(1, choice.cpu().long(), weight.cpu().double())
    full = torch.zeros(rows, experts, dtype=F64).scatter(1, want, shares)
    same = ((got > 0) == (full > 0)).all(-1)
    assert float((~same).float().mean()) <= 0.002  # two logits equal to within rounding, if any
    assert rel(got[same], full[same]) < 1e-5 and rel(gate, torch.sigmoid(z[:, experts])) < 1e-5
    assert torch.equal(counts.cpu(), torch.bincount(choice.cpu().flatten().long(), minlength=experts).int())
    ops.raise_on_error(CUDA)


def test_far_logits_still_share_by_a_softmax_of_the_chosen():
    """A logit some hundreds above the others: the others' scores vanish, and they are still chosen in their order."""
    router = torch.zeros(4, 8)
    bias = torch.tensor([-300.0, 100.0, -299.0, -301.0])
    choice, weight = ops.moe_route(torch.ones(1, 8, device=CUDA), router.to(CUDA), None, 4, 3, torch.zeros(4, dtype=torch.int32, device=CUDA),
                                   "chosen", bias=bias.to(CUDA))
    assert choice[0].tolist() == [1, 2, 0] and weight[0].tolist() == [1.0, 0.0, 0.0]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,hidden,inner,experts,top,shared", [(1, 64, 40, 6, 2, 24), (9, 100, 12, 5, 5, 36), (300, 64, 32, 7, 3, 64),
                                                                 (1500, 128, 96, 8, 4, 80), (17, 72, 56, 1, 1, 8), (3, 30, 7, 4, 2, 9)])
def test_ungated_experts_and_a_gated_shared_one(dtype, rows, hidden, inner, experts, top, shared):
    """Each form of the grouped products (ordinary cores, mma.sync, tcgen05) through the part itself."""
    part = RoutedExperts(hidden, inner, experts, top, correction=False, scoring="chosen", shared_inner=shared, router_bias=True,
                         unit="gelu_erf", shared_gate=True)
    W = draw(part, rows, {f"e{e}.up": 1.5 for e in range(experts)} | {"shared.up": 1.5, "router": 2.0, "router.b": 0.5})
    part = loaded(part, W, dtype)
    h = torch.randn(rows, hidden, generator=torch.Generator().manual_seed(rows)).to(DTYPES[dtype])
    got = part.forward(h.to(CUDA), LayerContext(Batch([rows]), None, None, 0)).cpu().double()
    want = plain.experts(h.to(F64), W, "", {"router": {"experts": experts, "top": top}, "shared": {"ff": shared}})
    err = (got - want).abs().amax(-1) / want.abs().max()
    assert int((err > (2e-5 if dtype == "float32" else 2e-2)).sum()) <= (rows // 500 if top < experts else 0)
    ops.raise_on_error(CUDA)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,hidden,inner", [(1, 64, 40), (16, 96, 56), (50, 72, 24), (3, 100, 36), (400, 128, 264), (700, 256, 640)])
def test_the_two_gelus_in_and_behind_the_products(dtype, rows, hidden, inner):
    g = torch.Generator().manual_seed(rows + hidden)
    dt = DTYPES[dtype]
    h = torch.randn(rows, hidden, generator=g).to(dt)
    part = GLUMLP(hidden, inner, "gelu_tanh")
    W = draw(part, rows, {"gate": 3.0})
    part = loaded(part, W, dtype)
    tol = 1e-5 if dtype == "float32" else 1.5e-2
    assert rel(part.forward(h.to(CUDA), None), plain.dense(h.to(F64), W, "")) < tol
    up = (torch.randn(inner, hidden, generator=g) * 3 * hidden ** -0.5).to(dt)
    assert rel(ops.linear_act(h.to(CUDA), up.to(CUDA), "gelu_erf"), plain.gelu_erf(h.to(F64) @ up.to(F64).T)) < tol
    z = torch.linspace(-9, 9, 400, device=CUDA)[None]
    assert rel(ops.activation(z, "gelu_erf"), plain.gelu_erf(z.cpu().to(F64))) < 1e-6


@pytest.mark.parametrize("rows", [1, 5, 8])
def test_a_pending_residual_step_in_front_of_the_gated_unit(rows):
    """The residual step and norm run inside the first product, the tanh form of GELU in its epilogue."""
    hidden, inner, eps = 128, 96, 1e-5
    part = GLUMLP(hidden, inner, "gelu_tanh")
    W = draw(part, 3, {"gate": 2.0})
    part = loaded(part, W, "bfloat16")
    g = torch.Generator().manual_seed(rows)
    x, branch, w = torch.randn(rows, hidden, generator=g), torch.randn(rows, hidden, generator=g).to(torch.bfloat16), 1 + 0.1 * torch.randn(hidden, generator=g)
    pending = ops.PendingStep(x.to(CUDA), branch.to(CUDA), None, None, w.to(CUDA), eps)
    got = part.forward(pending, None)
    new = x.double() + branch.double()
    assert rel(ops.residual_after(pending, None), new) < 1e-6
    assert rel(got, plain.dense(plain.rms(new, eps, w), W, "")) < 2e-2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [1, 8, 16, 50, 400])
def test_a_product_that_stays_in_float32(dtype, rows):
    """Unrounded on every path, also with a pending residual step in front: far closer than one bfloat16 rounding."""
    g = torch.Generator().manual_seed(rows)
    h, w = torch.randn(rows, 128, generator=g).to(DTYPES[dtype]), (torch.randn(72, 128, generator=g) * 128 ** -0.5).to(DTYPES[dtype])
    got = ops.linear_wide(h.to(CUDA), w.to(CUDA))
    assert got.dtype == torch.float32 and rel(got, h.double() @ w.double().T) < 1e-5
    if dtype == "bfloat16" and rows <= 8:
        x, nw = torch.randn(rows, 128, generator=g), 1 + 0.1 * torch.randn(128, generator=g)
        pending = ops.PendingStep(x.to(CUDA), h.to(CUDA), None, None, nw.to(CUDA), 1e-5)
        got = ops.linear_wide(pending, w.to(CUDA))
        normed = plain.rms(x.double() + h.double(), 1e-5, nw).float().to(torch.bfloat16).double()
        assert got.dtype == torch.float32 and rel(got, normed @ w.double().T) < 2e-3
        assert rel(ops.residual_after(pending, None), x.double() + h.double()) < 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens,width,stride", [(3, 64, 64), (5, 130, 139), (1, 7, 9), (40, 1024, 1200)])
def test_gating_rows_in_place(dtype, tokens, width, stride):
    g = torch.Generator().manual_seed(width)
    out, wide = torch.randn(tokens, width, generator=g).to(DTYPES[dtype]), torch.randn(tokens, stride, generator=g).to(DTYPES[dtype])
    gate = wide.to(CUDA)[:, stride - width:]
    got = ops.gate_rows(out.to(CUDA), gate)
    assert rel(got, out.double() * torch.sigmoid(wide[:, stride - width:].double())) < (1e-6 if dtype == "float32" else 6e-3)


# ---- the engine -----------------------------------------------------------------------------


def engine_for(name, dtype="float32", page=4, tokens=1024, requests=4, graphs=True, seed=0, raw=None):
    raw = raw or gc.config(name)
    weights = gc.tensors(raw, seed)
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


@pytest.mark.parametrize("name", sorted(gc.CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts(name, dtype):
    raw, weights, engine = engine_for(name, dtype)
    for n in (1, 2, 3, 41, 230):
        ids = gc.prompt(n, raw["vocab"], n)
        request = engine.cache.open("r")
        got = engine.runner.run([StepEntry(request, ids, list(range(n)))])
        engine.cache.close("r")
        assert_rows(got, plain.forward(ids, weights, raw), dtype, n, strict=every_expert(raw))
    ops.raise_on_error(CUDA)


@pytest.mark.parametrize("name,page", [("G", 4), ("H", 16), ("J", 8)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_decoding_and_mixed_batches(tmp_path, name, page, dtype):
    """Six requests over four state slots: prompts read whole, in portions of 2 to 9 tokens and
    token by token, decoded tokens beside portions of other requests, requests that end and whose
    pages and slots the next ones take (free pages are filled with NaN before every step)."""
    raw, weights, engine = engine_for(name, dtype, page=page, tokens=448)
    V = raw["vocab"]
    ids = {r: gc.prompt(n, V, i) for i, (r, n) in enumerate({"a": 170, "b": 33, "c": 2, "d": 58, "e": 60, "f": 17}.items())}
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


@pytest.mark.parametrize("name", sorted(gc.CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_equals_decoding_token_by_token(name, dtype):
    """The same prompt whole, and one token a step (captured decode steps, and launched one by one)."""
    for graphs in (True, False):
        raw, weights, engine = engine_for(name, dtype, graphs=graphs)
        ids = gc.prompt(75, raw["vocab"], 77)
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
    raw, weights, engine = engine_for("H", dtype, page=16, tokens=1024)
    ids = gc.prompt(700, raw["vocab"], 5)
    ids[-1] = ids[11]
    other = gc.prompt(50, raw["vocab"], 6)
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
    raw, weights, engine = engine_for("G", "float32")
    ids = gc.prompt(80, raw["vocab"], 8)
    request = engine.cache.open("r")
    got = [engine.runner.run([StepEntry(request, ids[:50], list(range(50)))])]
    got += [engine.runner.run([StepEntry(request, [t], [0])]) for t in ids[50:]]
    expect = plain.forward(ids, weights, raw)
    assert rel(torch.cat(got), expect) < TOLERANCE["float32"]

    def moved(change, w=weights):
        other = gc.config("G")
        change(other["layers"])
        out = plain.forward(ids, w, other)
        return min(rel(out[:50], expect[:50]), rel(out[50:], expect[50:]))

    assert moved(lambda l: l[0]["mixer"].update(scale=0.35)) > 1e-3
    assert moved(lambda l: l[0]["mixer"]["mask"].update(size=12)) > 1e-3
    assert moved(lambda l: l[0]["mixer"]["mask"].update(keep_first=4)) > 1e-3
    assert moved(lambda l: l[5]["mixer"]["mask"].update(keep_first=2)) > 1e-3
    assert moved(lambda l: l[0]["mixer"].update(v_mix=False)) > 1e-3
    assert moved(lambda l: l[5]["mixer"].update(v_mix=False)) > 1e-3
    assert moved(lambda l: l[1]["mixer"].update(norm_groups=1)) > 1e-3
    assert moved(lambda l: l[3]["mixer"].update(scale=0.25)) > 1e-3
    assert moved(lambda l: l[3]["mixer"]["mask"].update(size=10)) > 1e-3
    assert moved(lambda l: l[3]["mixer"]["rot"].update(base=1000.0)) > 1e-3
    assert moved(lambda l: l[3]["mlp"]["router"].update(top=3)) > 1e-3
    for name in ("l1.mix.dt_bias", "l1.mix.A_log", "l1.mix.D", "l1.mix.conv.b", "l4.mix.vmix", "l0.mlp.router.b", "l3.mlp.shared.sg"):
        other = weights[name].clone()
        other.view(-1)[0] += 0.3
        assert moved(lambda l: None, {**weights, name: other}) > 1e-3, name


WINDOWS = [("attention", 9, 0, 4, 16), ("attention", 16, 5, 16, 64), ("attention", 33, 16, 16, 64), ("attention", 1, 3, 4, 32),
           ("attention", 7, 17, 8, 128), ("latent_attention", 9, 0, 4, 16), ("latent_attention", 16, 0, 16, 64),
           ("latent_attention", 33, 0, 8, 64), ("latent_attention", 1, 0, 4, 64)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,window,keep,page,width", WINDOWS)
def test_a_token_enters_and_leaves_a_window(dtype, kind, window, keep, page, width):
    """One layer of windowed attention alone: a token changed at position p moves the logits of p to
    p + window - 1 and, to the last bit, of no other place (a kept one of every later place), in a prompt, in
    portions and in decoding, with pages given back behind the window."""
    if kind == "attention":
        mixer = {"heads": 4, "kv_heads": 2, "dim": width, "vdim": width, "scale": width ** -0.5, "mask": {"size": window, "keep_first": keep}}
    else:
        mixer = {"heads": 2, "dim": 16, "rot_dim": 32 if width % 64 == 0 else 8, "vdim": 24, "kv_rank": width, "scale": 0.2,
                 "mask": {"size": window}, "rot": {"base": 100.0, "dims": 32 if width % 64 == 0 else 8}}
    raw = {"architecture": "Gisudra", "vocab": 97, "width": 64, "norm": {"eps": 1e-6}, "layers": [{"type": kind, "mlp": None, "mixer": mixer}]}
    weights = gc.tensors(raw, 1)
    engine = Engine.from_tensors(raw, weights, EngineArgs(dtype=dtype, page_size=page, cache_tokens=256, max_requests=2,
                                                          cuda_graphs=False))  # one plan for equal steps: bits are compared
    ids = gc.prompt(90, 97, 3)

    def run(tokens, cuts):
        request, out, at = engine.cache.open("r"), [], 0
        for n in cuts:
            poison_free_pages(engine)
            out.append(engine.runner.run([StepEntry(request, tokens[at: at + n], list(range(n)))]).cpu())
            at += n
        engine.cache.close("r")
        return torch.cat(out)

    for cuts in ([90], [20, 2, 19, 9, 40], [42] + [1] * 48):
        base = run(ids, cuts)
        assert_rows(base, plain.forward(ids, weights, raw), dtype, strict=True)
        for p in [41, keep] + ([keep - 1] if keep else []):
            other = list(ids)
            other[p] = (other[p] + 1) % 97
            changed = ((base - run(other, cuts)).abs().amax(-1) > 0).nonzero().flatten().tolist()
            expected = list(range(p, 90 if p < keep else min(p + window, 90)))
            if dtype == "float32":
                assert changed == expected, (cuts[:3], p)
            else:  # a small change may vanish where a row is rounded to 16 bits
                assert set(changed) <= set(expected) and len(changed) > 0.8 * len(expected), (cuts[:3], p)
    ops.raise_on_error(CUDA)


def test_layers_without_pages_and_a_model_of_one_recurrence():
    """Nothing in the paged cache at all: states only, through the same cache manager and captured steps."""
    raw = {"architecture": "Gisudra", "vocab": 64, "width": 40, "norm": {"eps": 1e-5},
           "layers": [{"type": "mamba2", "mlp": None, "mixer": {"heads": 4, "vdim": 12, "state": 20, "groups": 2, "conv": 3, "norm_groups": 4}},
                      {"type": "mamba2", "mlp": {"kind": "dense", "ff": 16},
                       "mixer": {"heads": 2, "vdim": 16, "state": 8, "groups": 1, "conv": 4, "norm_groups": 1}}]}
    weights = gc.tensors(raw, 2)
    engine = Engine.from_tensors(raw, weights, EngineArgs(dtype="float32", page_size=4, cache_tokens=64, max_requests=2))
    ids = gc.prompt(60, 64, 4)
    request = engine.cache.open("r")
    got = [engine.runner.run([StepEntry(request, ids[:23], list(range(23)))])]
    got += [engine.runner.run([StepEntry(request, [t], [0])]) for t in ids[23:]]
    assert_rows(torch.cat(got), plain.forward(ids, weights, raw), "float32")


def test_greedy_generation_long_decoding_and_the_scheduler(tmp_path):
    """Through `load(...).generate`: the scheduler admits, batches and chunks; greedy ids are the plain
    implementation's best, 200 tokens past a two-token prompt included (the states are carried through
    all of them)."""
    raw = gc.config("G")
    weights = gc.tensors("G", 3)
    folder = tmp_path / "m"
    gc.write_folder(folder, raw, weights)
    model = load(folder, dtype="float32", page_size=8, cache_tokens=1024, max_requests=4, max_tokens_per_step=16)
    prompts = [gc.prompt(n, raw["vocab"], 20 + n) for n in (2, 5, 23, 40, 9, 31)]
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

    raw = gc.config("H")
    folder = write_random_model(tmp_path / "m", raw, seed=4)
    weights = {k: v.float() for k, v in load_file(str(folder / "model.safetensors")).items()}
    ids = gc.prompt(90, raw["vocab"], 1)
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
