"""Saralix on a GPU against the plain implementation: each added kernel alone, then the engine -- the
residual stream layer by layer, whole prompts, the tail one token at a time, prompts in portions down
to two tokens, batches of unequal requests whose shorter ones end earlier (slots, pages and states used
again), a far key among hundreds, across page borders and just inside and just outside a window in
prompts, portions and decoding, the first tokens, long decoding through the captured decode step,
greedy generation through the entry point, and the trace replay program."""
import json
import os

import pytest
import torch
import torch.nn.functional as F

from plain_saralix import (attend, causal_conv, clamped_glu, layer_norm, over_rms, rotate_halves, route, ssm_scan,
                           visible, yarn)
from saralix_helpers import (CONFIGS, NEEDLE, TOL, add_portions, needle_model, needle_tokens, plain_generate_greedy,
                             plain_logits, random_tokens, safe_tokens, weights_of, yarn_scaling)
from trace_tools import (Trace, add_batches, add_tail, add_whole, compare, forced_decode, run_in_process,
                         run_trace_run)

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16", "float16"]
LOOSE = {torch.float32: 2e-5, torch.bfloat16: 2e-2, torch.float16: 3e-3}


@pytest.fixture(scope="module")
def ops():
    from yalm_b200.csrc import ops as o
    o.lib()
    return o


class B:
    """The index arrays of a ragged batch."""

    def __init__(self, q_lens, slots):
        qs = [0]
        for q in q_lens:
            qs.append(qs[-1] + q)
        self.n_seqs, self.n_tokens, self.q_lens, self.slots = len(q_lens), qs[-1], q_lens, slots
        self.is_decode = all(q == 1 for q in q_lens)
        self.q_start = torch.tensor(qs, dtype=torch.int32, device=DEV)
        self.seq_slot = torch.tensor(slots, dtype=torch.int32, device=DEV)
        self.token_seq = torch.tensor(sum([[i] * q for i, q in enumerate(q_lens)], []), dtype=torch.int32, device=DEV)


def _lm(cfg, w, dtype, **kw):
    from yalm_b200 import LM
    from yalm_b200.config import config_from_dict
    return LM(config_from_dict(cfg), dict(w), dtype=dtype, **kw)


def close(got, ref, tol):
    return (got.double().cpu() - ref.double()).abs().max().item() <= tol * max(1e-6, ref.abs().max().item())


def rnd_of(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *shape: torch.randn(*shape, generator=g, dtype=torch.float64)


dev = lambda t: t.float().to(DEV)


# ------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dim, rows", [(64, 5), (100, 3), (1000, 70), (2048, 520), (4100, 2), (30, 4), (9000, 3), (4, 600)])
def test_layer_norm_form(ops, dim, rows):
    """As the norm of an output, as the norm of the stream, and both in one step; beside the other forms;
    rows with a large mean, whose deviations alone the variance is made of."""
    rnd = rnd_of(dim)
    x, a, w1, w2 = rnd(rows, dim) + 30.0, rnd(3, rows, dim) - 5.0, rnd(dim), rnd(dim)
    layer = lambda w: (ops.NORM_LAYER, dev(w), None, 0.0, 1e-5)
    rms = (ops.NORM_RMS, dev(w2), None, 0.0, 1e-5)
    y = 0.7 * a.sum(0)
    forms = {"layer": (layer(w2), lambda v: layer_norm(v, w2, 1e-5)), "rms": (rms, lambda v: over_rms(v, 1e-5) * w2),
             "none": ((ops.NORM_NONE, None, None, 0.0, 0.0), lambda v: v)}
    new = x + layer_norm(y, w1, 1e-5)
    for pre, (form, f) in forms.items():
        for dt in (torch.float32, torch.bfloat16):
            xd, h = dev(x), torch.empty(rows, dim, dtype=dt, device=DEV)
            ops.norm_step(xd, [(dev(a), 3, 0.7)], post=layer(w1), pre=form, h=h)
            assert close(xd, new, 2e-6), pre
            assert close(h, f(new), 1e-4 if dt == torch.float32 else 1e-2), pre
    xd, h = dev(x), torch.empty(rows, dim, device=DEV)
    ops.norm_step(xd, [(dev(a), 3, 0.7)], post=rms, pre=layer(w1), h=h)
    ref = x + over_rms(y, 1e-5) * w2
    assert close(xd, ref, 2e-6) and close(h, layer_norm(ref, w1, 1e-5), 1e-4)
    want = torch.tensor([rows - 1, 0], dtype=torch.int32, device=DEV)
    h = torch.empty(2, dim, device=DEV)
    ops.norm_step(dev(x), pre=layer(w1), h=h, rows=want, n_rows=2)
    assert close(h, layer_norm(x, w1, 1e-5)[[rows - 1, 0]], 1e-4)


@pytest.mark.parametrize("taps, channels", [(2, 8), (4, 100), (8, 36), (3, 2052)])
def test_convolution_of_many_tokens(ops, taps, channels):
    """Steps of more than a thousand tokens in one slice (four channels per thread), sequences that start
    anywhere in a thread's run, one token among many, then portions on top."""
    rnd = rnd_of(taps * 100 + channels)
    w, bias = rnd(channels, taps), rnd(channels)
    state = torch.zeros(5, taps - 1, channels, device=DEV)
    before = {s: torch.zeros(taps - 1, channels, dtype=torch.float64) for s in range(5)}
    for q_lens, slots in [([700, 1, 2, 403], [4, 0, 2, 1]), ([1, 1100], [4, 3]), ([5, 1, 1090], [0, 2, 4]), ([1, 1], [4, 2])]:
        b = B(q_lens, slots)
        src = rnd(1, b.n_tokens, channels + 12)
        out = torch.zeros(b.n_tokens, channels + 4, device=DEV)
        ops.short_conv(dev(src), 1, 8, channels, dev(w), state, b, out32=out, out_col0=4, out_bias=dev(bias), silu=True)
        at = 0
        for ql, s in zip(q_lens, slots):
            y, before[s] = causal_conv(src[0, at:at + ql, 8:8 + channels], w, bias, before[s])
            assert close(out[at:at + ql, 4:], F.silu(y), 1e-5), (q_lens, s)
            assert close(state[s], before[s], 1e-6), (q_lens, s)
            at += ql


# heads, heads per group, value size, state size
@pytest.mark.parametrize("H, G, P, N", [(4, 2, 24, 40), (1, 1, 64, 128), (3, 3, 10, 21), (6, 1, 33, 64), (2, 1, 70, 256),
                                        (8, 4, 32, 130), (2, 2, 8, 4)])
def test_state_space_scan(ops, H, G, P, N):
    """Unequal sequences with a carried state; decays from 0.9999 per token to almost nothing, steps small
    and large, in one sequence and across runs of tokens; one token at a time the same; other slots untouched."""
    rnd = rnd_of(H * 1000 + N)
    inner, row = H * P, H * P + 2 * G * N
    a_log = torch.linspace(-7.0, 3.0, H, dtype=torch.float64)
    bias, skip = rnd(H) - 1.0, rnd(H)
    q_lens, slots = [45, 1, 18, 203], [2, 0, 3, 5]
    b = B(q_lens, slots)
    n = b.n_tokens
    act, raw = rnd(n, row), 2.0 * rnd(2, n, H + 3)
    S0 = 0.3 * rnd(6, H, N, P)
    kept = S0.transpose(2, 3).contiguous().float().to(DEV)                     # the library's layout: [H, P, N]
    state, out = kept.clone(), torch.empty(n, inner, device=DEV)
    args = (dev(bias), dev(a_log), dev(skip))
    ops.ssd_scan(dev(act), dev(raw), 2, 3, *args, b, state, out, H, G, P, N)
    dt = F.softplus(raw.sum(0)[:, 3:] + bias)
    x, Bm, Cm = act[:, :inner].view(n, H, P), act[:, inner:inner + G * N].view(n, G, N), act[:, inner + G * N:].view(n, G, N)
    at = 0
    for ql, s in zip(q_lens, slots):
        for h in range(H):
            S, g = S0[s, h].clone(), h // (H // G)
            ref = ssm_scan(x[at:at + ql, h], Bm[at:at + ql, g], Cm[at:at + ql, g], dt[at:at + ql, h], a_log[h], skip[h], S)
            assert close(out[at:at + ql].view(ql, H, P)[:, h], ref, 2e-5), (s, h)
            assert close(state[s, h].T, S, 2e-5), (s, h)
        at += ql
    assert torch.equal(state[1], kept[1]) and torch.equal(state[4], kept[4])
    # token by token (the one-token kernel) from the same start
    step_state, at = kept.clone(), [0, 45, 46, 64]
    for t in range(18):
        live = [i for i, ql in enumerate(q_lens) if t < ql]
        bt = B([1] * len(live), [slots[i] for i in live])
        rows = torch.tensor([at[i] + t for i in live])
        o = torch.empty(len(live), inner, device=DEV)
        ops.ssd_scan(dev(act[rows]), dev(raw[:, rows]), 2, 3, *args, bt, step_state, o, H, G, P, N)
        assert close(o, out[rows.to(DEV)].cpu(), 2e-5), t
    assert close(step_state[3], state[3].cpu(), 2e-5)


def test_a_state_that_is_nearly_forgotten(ops):
    """A huge state followed by decays down to exp(-15) over a run of tokens or in one token, and tiny inputs:
    what is left is the inputs', not the difference of two roundings of the old state."""
    H, G, P, N, n = 1, 1, 4, 8, 24
    rnd = rnd_of(8)
    act, raw = 1e-3 * rnd(n, P + 2 * N), torch.zeros(1, n, 1, dtype=torch.float64)
    for log_a in (0.0, 1.0, 3.1, 5.0):
        a_log, bias, skip = torch.tensor([log_a]).double(), torch.tensor([0.0]).double(), torch.tensor([0.0]).double()
        for pieces in ([n], [1] * n):
            S, state, at = 1e4 * torch.ones(N, P, dtype=torch.float64), 1e4 * torch.ones(1, H, P, N, device=DEV), 0
            for k in pieces:
                out = torch.empty(k, P, device=DEV)
                ops.ssd_scan(dev(act[at:at + k]), dev(raw[:, at:at + k]), 1, 0, dev(bias), dev(a_log), dev(skip), B([k], [0]),
                             state, out, H, G, P, N)
                at += k
            ref = ssm_scan(act[:, :P], act[:, P:P + N], act[:, P + N:], F.softplus(raw[0, :, 0]), a_log[0], skip[0], S)
            assert close(state[0, 0].T, S, 5e-5) and close(out[-1], ref[-1], 5e-5), (log_a, len(pieces))


def test_long_lived_states_do_not_drift(ops):
    """Decays of 0.9997 over three thousand tokens, whole and one token at a time: the state stays as close to
    64-bit arithmetic as its own roundings allow."""
    H, G, P, N, n = 1, 1, 4, 8, 3000
    rnd = rnd_of(3)
    act, raw = rnd(n, P + 2 * N).abs(), torch.zeros(1, n, 1, dtype=torch.float64)
    a_log, bias, skip = torch.tensor([-7.7]).double(), torch.tensor([0.0]).double(), torch.tensor([0.0]).double()
    S = torch.zeros(N, P, dtype=torch.float64)
    ref = ssm_scan(act[:, :P], act[:, P:P + N], act[:, P + N:], F.softplus(raw[0, :, 0]), a_log[0], skip[0], S)
    for pieces in ([n], [1] * n):
        state, at = torch.zeros(1, H, P, N, device=DEV), 0
        for k in pieces:
            out = torch.empty(k, P, device=DEV)
            ops.ssd_scan(dev(act[at:at + k]), dev(raw[:, at:at + k]), 1, 0, dev(bias), dev(a_log), dev(skip), B([k], [0]),
                         state, out, H, G, P, N)
            at += k
        assert close(state[0, 0].T, S, 5e-6), len(pieces)
        assert close(out[-1], ref[-1], 5e-6)


@pytest.mark.parametrize("inner, groups", [(64, 1), (120, 5), (90, 2), (4096, 8), (30, 30)])
def test_gated_group_norm(ops, inner, groups):
    rnd = rnd_of(inner + groups)
    y, z, w = rnd(7, inner), rnd(3, 7, inner + 10), rnd(inner)
    ref = y * F.silu(z.sum(0)[:, 6:6 + inner] if inner % 4 else z.sum(0)[:, 4:4 + inner])
    ref = over_rms(ref.view(7, groups, -1), 1e-5).reshape(7, inner) * w
    for dt in (torch.float32, torch.bfloat16):
        out = torch.empty(7, inner, dtype=dt, device=DEV)
        ops.gated_group_norm(dev(y), dev(z), 3, 6 if inner % 4 else 4, dev(w), out, groups, 1e-5)
        assert close(out, ref, 1e-5 if dt == torch.float32 else 1e-2)


def test_weighted_sum_without_the_stream(ops):
    rnd = rnd_of(1)
    for dim in (32, 30):
        y, w = rnd(12, dim), rnd(4, 3)
        rows = torch.randperm(12, generator=torch.Generator().manual_seed(2)).to(torch.int32)
        x = torch.full((4, dim), 7.0, device=DEV)
        ops.routed_combine(x, dev(y), rows.to(DEV), dev(w).view(-1), 3, accumulate=False)
        ref = (y[rows.long()].view(4, 3, dim) * w[:, :, None]).sum(1)
        assert close(x, ref, 1e-6)
        ops.routed_combine(x, dev(y), rows.to(DEV), dev(w).view(-1), 3)
        assert close(x, 2 * ref, 1e-6)


def test_softmax_over_the_chosen_logits(ops):
    """The routing rule as the design states it, against the library's (softmax over all, divided by the
    chosen ones' sum), with logits far apart too."""
    g = torch.Generator().manual_seed(5)
    for E, top, spread in ((6, 2, 2.0), (3, 1, 1.0), (64, 6, 2.0), (5, 5, 1.0), (16, 4, 30.0)):
        n = 40
        z = spread * torch.randn(1, n, E, generator=g, dtype=torch.float64)
        choice, weight = torch.empty(n * top, dtype=torch.int32, device=DEV), torch.empty(n * top, device=DEV)
        counts = torch.zeros(E, dtype=torch.int32, device=DEV)
        ops.route_topk(dev(z), 1, n, E, 1, 1, top, True, choice, weight, counts)
        choice, weight = choice.cpu().view(n, top), weight.cpu().view(n, top)
        for t in range(n):
            chosen, w, margin = route(z[0, t], top)
            if margin > 1e-4:
                assert choice[t].tolist() == chosen.tolist() and close(weight[t], w, 2e-5), (E, t)


class LatentCase:
    """Random queries and latent rows of a few sequences, and the plain attention over them."""

    def __init__(self, seed, H, dim, rd, vdim, rank, window, dt, scale=0.3, sinks=True):
        rnd = rnd_of(seed)
        self.H, self.dim, self.rd, self.vdim, self.rank, self.window, self.scale, self.dt = H, dim, rd, vdim, rank, window, scale, dt
        self.hd = -(-(rank + rd) // 16) * 16
        r = lambda t: t.to(dt).double()                                     # values the storage type holds exactly
        self.uk, self.uv = r(rnd(H, dim, rank) * rank ** -0.5), r(rnd(H, vdim, rank) * rank ** -0.5)
        self.sink = 2.0 * rnd(H) if sinks else None
        self.rnd, self.r = rnd, r

    def sequence(self, n):
        """(q [n, H, dim + rd] rotated, c [n, rank], kr [n, rd])"""
        return self.rnd(n, self.H, self.dim + self.rd), self.r(self.rnd(n, self.rank)), self.r(self.rnd(n, self.rd))

    def reference(self, q, c, kr, first):
        """Outputs of the queries from position ``first`` on."""
        K = c.shape[0]
        k = torch.cat([torch.einsum("kr,hdr->khd", c, self.uk), kr[:, None].expand(K, self.H, self.rd)], -1)
        v = torch.einsum("kr,hdr->khd", c, self.uv)
        return attend(q[first:], k, v, visible(K - first, first, self.window), self.scale, self.sink)

    def rows(self, c, kr):
        """[n, 2, 1, hd] as the library keeps a step's rows"""
        row = torch.zeros(c.shape[0], self.hd, dtype=torch.float64)
        row[:, :self.rank], row[:, self.rank:self.rank + self.rd] = c, kr
        return row[:, None, None].expand(-1, 2, 1, -1).to(self.dt).to(DEV).contiguous()

    def absorbed(self, q):
        out = torch.zeros(q.shape[0], self.H, self.hd, dtype=torch.float64)
        out[..., :self.rank] = torch.einsum("thd,hdr->thr", q[..., :self.dim], self.uk)
        out[..., self.rank:self.rank + self.rd] = q[..., self.dim:]
        return out.to(self.dt).to(DEV).view(q.shape[0], -1).contiguous()


LATENT_SHAPES = [(3, 24, 8, 16, 40, 33), (20, 16, 16, 24, 72, None), (1, 48, 24, 64, 200, 64), (5, 10, 2, 12, 21, 7),
                 (4, 32, 16, 40, 300, None), (17, 16, 64, 32, 512, 100), (2, 8, 0, 16, 64, 1), (2, 16, 16, 16, 600, None)]


@pytest.mark.parametrize("H, dim, rd, vdim, rank, window", LATENT_SHAPES)
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16, torch.float16])
def test_absorbed_attention_and_expansion(ops, H, dim, rd, vdim, rank, window, dt):
    """Decode steps and portions over a cache with and without pages, rings that have wrapped, one run of keys
    per query and several (some of them empty), sinks of the scores' size, with both kernels and both kinds of gate."""
    case = LatentCase(rank + H, H, dim, rd, vdim, rank, window, dt)
    cap = window or 320
    lens, slots = [1, 200, 31, 129], [2, 0, 3, 1]
    seqs = [case.sequence(n) for n in lens]
    for q_lens in ([1, 1, 1, 1], [1, 5, 2, 9]):
        past = [n - q for n, q in zip(lens, q_lens)]
        b = B(q_lens, slots)
        slot_pos = torch.zeros(4, dtype=torch.int32)
        plain_cache = torch.zeros(4, 1, cap, case.hd, dtype=dt, device=DEV)
        for (q, c, kr), s, p in zip(seqs, slots, past):
            slot_pos[s] = p
            rows = case.rows(c, kr)[:p, 0, 0]
            first = max(0, p - cap)
            plain_cache[s, 0, torch.arange(first, p, device=DEV) % cap] = rows[first:]
        pps = -(-cap // 64)
        pages = torch.randperm(4 * pps + 3, generator=torch.Generator().manual_seed(1))[:4 * pps].view(4, pps).to(torch.int32)
        paged = torch.zeros(1, 4 * pps + 3, 64, case.hd, dtype=dt, device=DEV)
        for s in range(4):
            for k in range(pps):
                piece = plain_cache[s, 0, 64 * k:64 * k + 64]
                paged[0, int(pages[s, k]), :piece.shape[0]] = piece
        slot_pos = slot_pos.to(DEV)
        kv_step = torch.cat([case.rows(c, kr)[p:] for (_, c, kr), p in zip(seqs, past)])
        q_abs = case.absorbed(torch.cat([q[p:] for (q, _, _), p in zip(seqs, past)]))
        ref = torch.cat([case.reference(q, c, kr, p) for (q, c, kr), p in zip(seqs, past)])
        n = b.n_tokens
        gate = {"head": case.rnd(2, n, H + 1), "element": case.rnd(2, n, H * vdim + 1)}
        uv = case.uv.transpose(1, 2).contiguous().to(dt).to(DEV)
        for mma in ([True, False] if dt != torch.float32 else [False]):
            for cache, table in ((plain_cache, None), (paged, pages.to(DEV))):
                for nsplit, per in ((1, 0), (3, 64), (9, 32), (2, 320)):
                    o_lat = torch.full((n, H * case.hd), 9.0, dtype=dt, device=DEV)
                    parts = None
                    if nsplit > 1:
                        parts = (torch.full((n, H, nsplit, rank), float("nan"), device=DEV),
                                 torch.full((n, H, nsplit, 2), float("nan"), device=DEV), nsplit)
                    ops.latent_attention(q_abs, kv_step, cache, b, slot_pos, o_lat if parts is None else None, H, rank, case.hd,
                                         cap, window, case.scale, sink=dev(case.sink), pages=table, parts=parts, mma=mma,
                                         per_split=per)
                    for mode, name in ((ops.GATE_NONE, None), (ops.GATE_HEAD, "head"), (ops.GATE_ELEMENT, "element")):
                        out = torch.empty(n, H * vdim, dtype=dt, device=DEV)
                        ops.latent_expand(o_lat, uv, dev(gate[name]) if name else None, 2, out, H, rank, vdim, case.hd,
                                          parts=parts, gate_col0=1, gate_mode=mode)
                        want = ref
                        if name:
                            z = torch.sigmoid(gate[name].sum(0)[:, 1:])
                            want = ref * (z[:, :, None] if name == "head" else z.view(n, H, vdim))
                        assert close(out.view(n, H, vdim), want, LOOSE[dt]), (q_lens, mma, table is not None, nsplit, name)


@pytest.mark.parametrize("H, dim, rd, vdim, rank, window", [s for s in LATENT_SHAPES if all(v % 8 == 0 for v in s[1:5])])
@pytest.mark.parametrize("dt", [torch.bfloat16, torch.float16])
def test_expanded_attention_of_whole_prompts(ops, H, dim, rd, vdim, rank, window, dt):
    case = LatentCase(rank + H + 1, H, dim, rd, vdim, rank, window, dt)
    assert ops.latent_prefill_usable(dt, dim, rd, vdim, rank, case.hd)
    lens = [1, 200, 64, 65, 31, 129]
    b = B(lens, [5, 0, 2, 1, 4, 3])
    seqs = [case.sequence(n) for n in lens]
    q = torch.cat([s[0] for s in seqs]).to(dt)
    c = torch.cat([s[1] for s in seqs])
    kv = torch.cat([torch.einsum("kr,hdr->khd", c, case.uk), torch.einsum("kr,hdr->khd", c, case.uv)], -1).to(dt).to(DEV)
    rows = torch.cat([case.rows(s[1], s[2]) for s in seqs])
    ref = torch.cat([case.reference(s[0], s[1], s[2], 0) for s in seqs])
    n = b.n_tokens
    gate = {None: None, "head": case.rnd(2, n, H + 1), "element": case.rnd(2, n, H * vdim + 1)}
    for mode, name in ((ops.GATE_NONE, None), (ops.GATE_HEAD, "head"), (ops.GATE_ELEMENT, "element")):
        out = torch.full((n, H * vdim), 9.0, dtype=dt, device=DEV)
        ops.latent_prefill(q.to(DEV).view(n, -1).contiguous(), kv.view(n, -1).contiguous(), rows, b, out, H, dim, rd, vdim, rank,
                           case.hd, window, case.scale, sink=dev(case.sink), gate=dev(gate[name]) if name else None, gate_n=2,
                           gate_col0=1, gate_mode=mode)
        want = ref
        if name:
            z = torch.sigmoid(gate[name].sum(0)[:, 1:])
            want = ref * (z[:, :, None] if name == "head" else z.view(n, H, vdim))
        assert close(out.view(n, H, vdim), want, LOOSE[dt]), name


@pytest.mark.parametrize("window", [None, 5, 64, 70])
@pytest.mark.parametrize("where", ["prompt", "decode"])
def test_one_key_at_the_edge_of_a_window(ops, window, where):
    """A key whose score stands far above all others, right inside and right outside a window and at page
    borders: it takes the whole weight or none of it; a sink above every score takes it all."""
    H, dim, rd, vdim, rank, dt = 2, 16, 8, 16, 32, torch.bfloat16
    case = LatentCase(7, H, dim, rd, vdim, rank, window, dt, scale=1.0)
    n = 150
    edges = sorted({p for p in (0, 1, 63, 64, 127, n - 2, n - 1, n - (window or n), n - (window or n) - 1) if 0 <= p < n})
    for loud in edges:
        q, c, kr = case.sequence(n)
        q, kr = 0.05 * q, 0.05 * kr
        kr[loud] = 0.0
        kr[loud, 0] = 8.0
        q[:, :, dim] = 4.0
        q, c, kr = q.to(dt).double(), c, kr.to(dt).double()
        for sink in (torch.full((H,), -3.0), torch.tensor([60.0, -3.0])):
            case.sink = sink.double()
            ref = case.reference(q, c, kr, 0 if where == "prompt" else n - 1)
            rows = case.rows(c, kr)
            if where == "prompt":
                b = B([n], [0])
                kv = torch.cat([torch.einsum("kr,hdr->khd", c, case.uk), torch.einsum("kr,hdr->khd", c, case.uv)], -1)
                out = torch.empty(n, H * vdim, dtype=dt, device=DEV)
                ops.latent_prefill(q.to(dt).to(DEV).view(n, -1).contiguous(), kv.to(dt).to(DEV).view(n, -1).contiguous(), rows, b, out,
                                   H, dim, rd, vdim, rank, case.hd, window, case.scale, sink=dev(case.sink))
            else:
                b, cap = B([1], [0]), window or 192
                cache = torch.zeros(1, 1, cap, case.hd, dtype=dt, device=DEV)
                first = max(0, n - 1 - cap)
                cache[0, 0, torch.arange(first, n - 1, device=DEV) % cap] = rows[first:n - 1, 0, 0]
                o_lat = torch.empty(1, H * case.hd, dtype=dt, device=DEV)
                out = torch.empty(1, H * vdim, dtype=dt, device=DEV)
                ops.latent_attention(case.absorbed(q[n - 1:]), rows[n - 1:], cache, b, torch.tensor([n - 1], dtype=torch.int32, device=DEV),
                                     o_lat, H, rank, case.hd, cap, window, case.scale, sink=dev(case.sink))
                ops.latent_expand(o_lat, case.uv.transpose(1, 2).contiguous().to(dt).to(DEV), None, 1, out, H, rank, vdim, case.hd)
            assert close(out.view(ref.shape), ref, 2e-2), (loud, sink.tolist())
            if sink[0] > 50:
                assert out.view(ref.shape)[-1, 0].abs().max() < 1e-3        # that head's weight is the sink's


@pytest.mark.parametrize("H, dim, rd, rank", [(3, 24, 8, 40), (2, 10, 2, 21), (5, 32, 64, 64), (1, 16, 12, 48)])
@pytest.mark.parametrize("halves", [True, False])
def test_rows_queries_and_rotation(ops, H, dim, rd, rank, halves):
    """The stored rows, the rotated and the absorbed queries, from columns of one stacked product in two
    slices: YaRN frequencies with a factor on cos and sin, pairs of halves and of neighbours, positions of
    two sequences far from zero; a step longer than a ring leaves the ring's last rows."""
    from yalm_b200.parts.position import yarn_frequencies
    rnd = rnd_of(dim + rd)
    scaling = yarn_scaling(8.0, 256)
    freqs, mult = yarn(rd, 1e4, scaling)
    f32, m32 = yarn_frequencies(rd, 1e4, scaling)
    assert m32 == pytest.approx(mult) and torch.allclose(f32.double(), freqs, rtol=1e-6)
    hd, cap, eps = -(-(rank + rd) // 16) * 16, 16, 1e-5
    lens, slots, starts = [21, 3], [1, 0], [500, 7]
    b = B(lens, slots)
    n, qd = b.n_tokens, dim + rd
    slot_pos = torch.tensor([7, 500], dtype=torch.int32, device=DEV)
    col_kv = H * qd
    src = rnd(2, n, col_kv + rank + rd + 3)
    z, w_c, uk = src.sum(0), 1.0 + 0.1 * rnd(rank), rnd(H, dim, rank)
    pos = torch.cat([torch.arange(s, s + q) for s, q in zip(starts, lens)])

    def turn(x):                                                   # [n, heads, rd]
        if halves:
            return rotate_halves(x, pos, freqs, mult)
        order = torch.cat([torch.arange(0, rd, 2), torch.arange(1, rd, 2)])
        out = torch.empty_like(x)
        out[..., order] = rotate_halves(x[..., order], pos, freqs, mult)
        return out

    both = z[:, col_kv:col_kv + rank + rd]
    c = over_rms(both[:, :rank], eps) * w_c
    kr = turn(both[:, None, rank:])[:, 0]
    q = z[:, :col_kv].view(n, H, qd)
    qr = turn(q[..., dim:])
    kw = {"halves": halves, "mult": mult}
    freq = f32.to(DEV)
    kv_step = torch.full((n, 2, 1, hd), 9.0, device=DEV)
    cache = torch.full((2, 1, cap, hd), 5.0, device=DEV)
    c_rows = torch.empty(n, rank, device=DEV)
    ops.latent_store(dev(src), 2, dev(w_c), eps, freq, b, slot_pos, kv_step, cache, rank, rd, hd, cap, col0=col_kv,
                     c_rows=c_rows, **kw)
    row = torch.cat([c, kr, torch.zeros(n, hd - rank - rd, dtype=torch.float64)], -1)
    assert close(kv_step[:, 0, 0], row, 1e-4) and torch.equal(kv_step[:, 0], kv_step[:, 1]) and torch.equal(c_rows, kv_step[:, 0, 0, :rank])
    at = 0
    for ql, s, p0 in zip(lens, slots, starts):
        for p in range(p0, p0 + ql):
            if p >= p0 + ql - cap:
                assert torch.equal(cache[s, 0, p % cap], kv_step[at + p - p0, 0, 0])
        at += ql
    assert int((cache[0, 0] == 5.0).all(-1).sum()) == cap - 3             # rows nobody wrote
    q_out = torch.empty(n, H * qd, device=DEV)
    ops.latent_rotate_q(dev(src), 2, freq, b, slot_pos, q_out, H, dim, rd, **kw)
    assert close(q_out.view(n, H, qd), torch.cat([q[..., :dim], qr], -1), 1e-4)
    ref = torch.cat([torch.einsum("thd,hdr->thr", q[..., :dim], uk), qr, torch.zeros(n, H, hd - rank - rd, dtype=torch.float64)], -1)
    for many in (1, 8):                                           # few tokens and many
        bb = b if many == 1 else B([l * many for l in lens], slots)
        s2 = src if many == 1 else rnd(2, bb.n_tokens, src.shape[-1])
        for dt in (torch.float32, torch.bfloat16):
            q_abs = torch.full((bb.n_tokens, H * hd), 9.0, dtype=dt, device=DEV)
            ops.latent_absorb_q(dev(s2), 2, uk.to(dt).to(DEV), freq, bb, slot_pos, q_abs, H, dim, rd, rank, hd, **kw)
            if many == 1:
                assert close(q_abs.view(n, H, hd), ref, 1e-4 if dt == torch.float32 else 2e-2)
            else:
                qq = s2.sum(0)[:, :col_kv].view(-1, H, qd)
                want = torch.einsum("thd,hdr->thr", qq[..., :dim], uk.to(dt).double())
                assert close(q_abs.view(-1, H, hd)[..., :rank], want, 1e-4 if dt == torch.float32 else 2e-2)


def test_clamped_feed_forward(ops):
    """The dense feed-forward as a part: inputs on both sides of the clamps, a width in pairs and one that is not."""
    from yalm_b200.parts import FEED_FORWARDS, ResidualStream, Runtime
    rnd = rnd_of(4)
    for dtype in (torch.float32, torch.bfloat16):
        rt = Runtime(dtype)
        for ff, n in ((48, 5), (50, 5), (64, 300)):
            part = FEED_FORWARDS["clamped_glu"]({"hidden_size": 40, "intermediate_size": ff, "limit": 1.25, "slope": 1.702,
                                                 "shift": 1.0}, rt)
            w = {k: rnd(*need.shape).to(torch.bfloat16) for k, need in part.tensor_needs().items()}
            part.bind(w)
            h = (0.3 * rnd(n, 40)).to(dtype)
            stream = ResidualStream(rt, torch.zeros(n, 40, device=DEV))
            part.forward(h.to(DEV), None, stream)
            d = {k: v.double() for k, v in w.items()}
            ref = clamped_glu(h.double() @ d["gate"].T, h.double() @ d["up"].T, 1.25) @ d["down"].T
            assert close(stream.resolve(), ref, 2e-5 if dtype == torch.float32 else 1e-2), (dtype, ff)


# ------------------------------------------------------------------ the engine
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_residual_stream_layer_by_layer(name):
    cfg, seed = CONFIGS[name]
    w = weights_of(name)
    toks, _ = safe_tokens(cfg, w, 90, seed + 5)
    want = []
    ref, _ = plain_logits(cfg, w, toks, taps=lambda i, x: want.append(x.clone()))
    for dtype, tol in (("float32", 2e-5), ("bfloat16", 4e-2)):
        lm = _lm(cfg, w, dtype, max_context=256, max_batch=2)
        got = []
        lm.model.tap = lambda i, stream: got.append(stream.total().double().cpu())
        logits = lm.step([toks], lm.acquire(1), [list(range(len(toks)))])
        lm.model.tap = None
        assert len(got) == len(want) == len(cfg["layers"])
        for i, (a, b) in enumerate(zip(got, want)):
            assert close(a, b, tol), f"{dtype}: the residual stream differs after layer {i}"
        assert close(logits, ref, TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_tail_portions_batches(name, dtype):
    cfg, seed = CONFIGS[name]
    w = weights_of(name)
    lengths = {"a": 150, "b": 1, "c": 66, "d": 23, "e": 129}           # across page borders (64, 128), one token
    reqs, refs = {}, {}
    for k, (rid, n) in enumerate(lengths.items()):
        reqs[rid], refs[rid] = safe_tokens(cfg, w, n, seed * 10 + k)
    tr = Trace()
    add_whole(tr, reqs)
    add_tail(tr, {r: reqs[r] for r in ("a", "c", "d")}, tail=40)
    for rid, sizes in (("a", [2, 3, 64, 2]), ("c", [63, 2]), ("d", [1, 2, 1, 5, 2, 2]), ("e", [64, 64])):
        add_portions(tr, rid, reqs[rid], sizes)
    # unequal requests together; the shorter end earlier; their slots and pages serve the next batch
    add_batches(tr, reqs, [["a", "b", "c"], ["d", "e", "b"], ["e", "a"]],
                {"a": 110, "b": 1, "c": 60, "d": 20, "e": 100})
    lm = _lm(cfg, w, dtype, max_context=256, max_batch=3, max_tokens=tr.max_tokens)
    compare(tr, run_in_process(lm, tr), refs, cfg["vocab"], TOL[dtype])


@pytest.mark.parametrize("window", [None, 40, 64, 130])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_needles_in_prompts_portions_and_decoding(dtype, window):
    cfg, w = needle_model(window)
    n, at = 420, 100
    edge = window or 200
    probes = sorted({p for p in (at + 1, 127, 128, at + edge - 2, at + edge - 1, at + edge, at + edge + 1, 319, 320, 419)
                     if p != at and p < n})
    toks = needle_tokens(n, [at], probes)
    ref, _ = plain_logits(cfg, w, toks)
    blind = list(toks)
    blind[at] = 9
    lost, _ = plain_logits(cfg, w, blind)
    for p in probes:                                      # a needle lost, or found outside the window, would show
        seen = window is None or p - at < window
        assert ((ref[p] - lost[p]).abs().max() > 0.4 * ref.abs().max()) == seen, p
    refs, reqs = {"n": ref, "s": ref[:at + edge + 3]}, {"n": toks, "s": toks[:at + edge + 3]}
    tr = Trace()
    add_whole(tr, {"n": toks})
    add_tail(tr, {"s": reqs["s"]}, tail=edge + 1)         # the needle, too, is decoded in some
    add_tail(tr, {"n": toks}, tail=110)
    add_portions(tr, "n", toks, [1, 62, 1, 2, 36, 2, 200])
    lm = _lm(cfg, w, dtype, max_context=512, max_batch=2, max_tokens=tr.max_tokens)
    compare(tr, run_in_process(lm, tr), refs, cfg["vocab"], TOL[dtype])
    # the needle as the sequence's very first token, the probe right after it
    first = needle_tokens(60, [0], [1, 39, 40, 59])
    ref0, _ = plain_logits(cfg, w, first)
    assert ref0[1].argmax() == NEEDLE
    tr = Trace()
    add_whole(tr, {"f": first})
    add_tail(tr, {"f": first}, tail=59)
    compare(tr, run_in_process(lm, tr), {"f": ref0}, cfg["vocab"], TOL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["sara_a", "sara_b"])
def test_long_decoding_through_the_captured_step(name, dtype):
    cfg, seed = CONFIGS[name]
    w = weights_of(name)
    reqs, refs = {}, {}
    for k, (rid, n) in enumerate({"x": 240, "y": 90, "z": 141}.items()):
        reqs[rid], refs[rid] = safe_tokens(cfg, w, n, seed * 7 + k)
    lm = _lm(cfg, w, dtype, max_context=256, max_batch=3)
    forced_decode(lm, reqs, {"x": 30, "y": 3, "z": 65}, refs, TOL[dtype])
    # the same slots again, other requests: nothing of the earlier states is left
    forced_decode(lm, reqs, {"x": 1, "y": 64, "z": 2}, refs, TOL[dtype], order=["z", "x", "y"])


def test_a_request_does_not_depend_on_its_batch():
    cfg, seed = CONFIGS["sara_a"]
    w = weights_of("sara_a")
    lens = {"a": 90, "b": 40, "c": 7, "d": 200}
    reqs = {r: random_tokens(n, cfg["vocab"], seed + k) for k, (r, n) in enumerate(lens.items())}
    lm = _lm(cfg, w, "float32", max_context=256, max_batch=4)
    alone = {}
    for r, t in reqs.items():
        s = lm.acquire(1)
        alone[r] = lm.step([t], s, [list(range(len(t)))]).cpu()
        lm.release(s)
    s = lm.acquire(4)
    both = lm.step([reqs[r] for r in reqs], s, [list(range(len(reqs[r]))) for r in reqs]).cpu()
    at = 0
    for r, t in reqs.items():
        assert close(both[at:at + len(t)], alone[r], 1e-6), r
        at += len(t)


def test_greedy_generation_through_the_entry_point():
    cfg, seed = CONFIGS["sara_a"]
    w = weights_of("sara_a")
    lm = _lm(cfg, w, "float32", max_context=128, max_batch=2)
    prompts = [random_tokens(9, cfg["vocab"], 1), random_tokens(45, cfg["vocab"], 2), random_tokens(2, cfg["vocab"], 3)]
    outs = lm.generate(prompts, max_new_tokens=12, temperature=0.0, ignore_eos=True)
    for p, o in zip(prompts, outs):
        assert list(o.tokens) == plain_generate_greedy(cfg, w, p, 12)


def write_model(path, cfg, w):
    from yalm_b200.weights import safetensors_io as st
    os.makedirs(path)
    with open(path / "config.json", "w") as f:
        json.dump(cfg, f)
    st.write_file(str(path / "model.safetensors"), w)


def test_trace_replay_program(tmp_path):
    cfg, seed = CONFIGS["sara_c"]
    w = weights_of("sara_c")
    write_model(tmp_path / "model", cfg, w)
    reqs, refs = {}, {}
    for k, (rid, n) in enumerate({"a": 70, "b": 9}.items()):
        reqs[rid], refs[rid] = safe_tokens(cfg, w, n, 50 + k)
    tr = Trace()
    add_whole(tr, reqs)
    add_tail(tr, reqs, tail=8)
    add_batches(tr, reqs, [["a", "b"]], {"a": 60, "b": 4})
    for dtype in ("bfloat16", "float32"):
        out = tmp_path / f"out_{dtype}"
        os.makedirs(out)
        got = run_trace_run(str(tmp_path / "model"), dtype, tr, str(out))
        compare(tr, got, refs, cfg["vocab"], TOL[dtype])


def test_command_line(tmp_path):
    """Writes a model folder of random weights for a configuration and generates from it."""
    import subprocess
    import sys
    from yalm_b200.weights import load_checkpoint
    cfg, _ = CONFIGS["sara_b"]
    with open(tmp_path / "cfg.json", "w") as f:
        json.dump(cfg, f)
    model = str(tmp_path / "model")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, "-m", "yalm_b200", model, "--dtype", "float32", "--random-weights",
                        str(tmp_path / "cfg.json"), "--seed", "3", "--tokens", "5,6,7;9,10", "-n", "6", "-t", "0"],
                       capture_output=True, text=True, cwd=root, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert "Saralix" in r.stdout
    lines = [l for l in r.stdout.splitlines() if l.startswith("tokens:")]
    w = load_checkpoint(model)
    for line, prompt in zip(lines, ([5, 6, 7], [9, 10])):
        assert [int(t) for t in line.split("(")[0].split()[1:]] == plain_generate_greedy(cfg, w, prompt, 6)
    assert len(lines) == 2
