"""Tetodra on a GPU against the plain implementation: each added kernel alone, then the engine -- the
residual stream layer by layer, whole prompts, the tail one token at a time, prompts in portions down
to two tokens, batches of unequal requests whose shorter ones end earlier (slots, pages and states used
again), a far key among hundreds, across page borders and at the edges of distance buckets in prompts,
portions and decoding, the first tokens, long decoding through the captured decode step, greedy
generation through the entry point, and the trace replay program."""
import json
import os

import pytest
import torch
import torch.nn.functional as F

from plain_tetodra import (attend, delta_rule, distance_bucket, gated_linear, layer_norm, matrix_memory,
                           over_rms, query_temperature, rotate_halves, unit)
from tetodra_helpers import (CONFIGS, NEEDLE, TOL, add_portions, needle_model, needle_tokens, plain_generate_greedy,
                             plain_logits, random_tokens, steady_tokens, weights_of)
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
def test_three_weighted_sets(ops, dim, rows):
    """The sum of up to three products, each with slices of its own, a factor, and a factor per feature or
    none; written alone, and together with each form of the next read."""
    rnd = rnd_of(dim)
    x = rnd(rows, dim)
    bufs = [rnd(s, rows, dim) for s in (3, 1, 9)]
    factors, weights = (0.7, -1.3, 0.4), (rnd(dim), None, rnd(dim))
    w = rnd(dim)
    none = (ops.NORM_NONE, None, None, 0.0, 0.0)
    forms = {"layer": ((ops.NORM_LAYER, dev(w), None, 0.0, 1e-5), lambda v: layer_norm(v, w, 1e-5)),
             "rms": ((ops.NORM_RMS, dev(w), None, 0.0, 1e-5), lambda v: over_rms(v, 1e-5) * w), "none": (none, lambda v: v)}
    for used in ([0], [0, 1], [2, 0, 1], [1, 2, 0]):
        sets = [(dev(bufs[k]), bufs[k].shape[0], factors[k]) + ((dev(weights[k]),) if weights[k] is not None else ())
                for k in used]
        new = x + sum(factors[k] * bufs[k].sum(0) * (1.0 if weights[k] is None else weights[k]) for k in used)
        xd = dev(x)
        ops.norm_step(xd, sets, post=none)
        assert close(xd, new, 2e-6), used
        for pre, (form, f) in forms.items():
            for dt in (torch.float32, torch.bfloat16):
                xd, h = dev(x), torch.empty(rows, dim, dtype=dt, device=DEV)
                ops.norm_step(xd, sets, post=none, pre=form, h=h)
                assert close(xd, new, 2e-6), (used, pre)
                assert close(h, f(new), 1e-4 if dt == torch.float32 else 1e-2), (used, pre)


def paged_copy(plain, pages, pps, size, dt):
    """A contiguous cache [slots, G, capacity, size] as pages [G, pages, 64, size]."""
    slots, G, cap, _ = plain.shape
    out = torch.zeros(G, slots * pps + 3, 64, size, dtype=dt, device=DEV)
    for s in range(slots):
        for k in range(pps):
            piece = plain[s, :, 64 * k:64 * k + 64]
            out[:, int(pages[s, k]), :piece.shape[1]] = piece
    return out


@pytest.mark.parametrize("H, G, dk, dv, true_dk, dims, has_v, norm", [
    (6, 2, 24, 40, 24, 16, True, False), (4, 2, 32, 32, 32, 0, False, True), (9, 1, 64, 128, 64, 0, True, False),
    (3, 3, 16, 16, 14, 6, True, False), (5, 5, 16, 16, 10, 0, False, True), (2, 1, 256, 200, 250, 250, True, True),
    (2, 1, 136, 136, 136, 64, False, True), (16, 4, 128, 256, 128, 128, True, False)])
def test_heads_are_normed_turned_and_stored(ops, H, G, dk, dv, true_dk, dims, has_v, norm):
    rnd = rnd_of(dk + dv + H)
    lens, slots, starts = [21, 3], [1, 0], [500, 7]
    b = B(lens, slots)
    n, cap, pps = b.n_tokens, 600, 10
    slot_pos = torch.tensor([7, 500], dtype=torch.int32, device=DEV)
    pages = torch.randperm(23, generator=torch.Generator().manual_seed(1))[:20].reshape(2, 10).to(torch.int32)
    row = H * dk + G * dk + (G * dv if has_v else 0)
    src = rnd(2, n, row)
    for h in range(H + G):                                        # features beyond a head's true size are zero
        src[:, :, h * dk + true_dk:(h + 1) * dk] = 0
    z = src.sum(0)
    pos = torch.cat([torch.arange(s, s + q) for s, q in zip(starts, lens)])
    w_q, w_k = torch.zeros(dk).double(), torch.zeros(dk).double()
    w_q[:true_dk], w_k[:true_dk] = 1.0 + 0.2 * rnd(true_dk), 1.0 + 0.2 * rnd(true_dk)
    q, k = z[:, :H * dk].view(n, H, dk), z[:, H * dk:(H + G) * dk].view(n, G, dk)
    v = z[:, (H + G) * dk:].view(n, G, dv) if has_v else k
    if norm:
        r = lambda x: 1.0 / torch.sqrt((x * x).sum(-1, keepdim=True) / true_dk + 1e-5)
        q, k = q * r(q) * w_q, k * r(k) * w_k
    q, k = rotate_halves(q, pos, dims, 1e4), rotate_halves(k, pos, dims, 1e4)
    temp = torch.tensor([query_temperature(int(p), 0.3, 6.0) for p in pos]).double()
    table = None
    if dims:
        freq = torch.tensor([1e4 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float32, device=DEV)
        table = torch.empty(n, dims // 2, 2, device=DEV)
        ops.rope_table(freq, b, slot_pos, table)
    for dt, tol in ((torch.float32, 1e-4), (torch.bfloat16, 1e-2)):
        for paged in (False, True):
            shape = (lambda size: (G, 23, 64, size)) if paged else (lambda size: (2, G, cap, size))
            kc, vc = (torch.full(shape(s), 5.0, dtype=dt, device=DEV) for s in (dk, dv))
            q_out = torch.full((n, H * dk), 9.0, dtype=dt, device=DEV)
            kv_step = torch.full((n, G * (dk + dv)), 9.0, dtype=dt, device=DEV)
            ops.head_store(dev(src), 2, (dev(w_q), dev(w_k), 1e-5, true_dk) if norm else None, table, dims, (0.3, 6.0), b,
                           slot_pos, q_out, kv_step, kc, vc, H, G, dk, dv, has_v, cap, pages=pages.to(DEV) if paged else None)
            assert close(q_out.view(n, H, dk), q * temp[:, None, None], tol)
            ks, vs = kv_step[:, :G * dk].view(n, G, dk), kv_step[:, G * dk:].view(n, G, dv)
            assert close(ks, k, tol) and close(vs, v, tol)
            at = 0
            for ql, s, p0 in zip(lens, slots, starts):
                for p in range(p0, p0 + ql):
                    place = (slice(None), int(pages[s, p // 64]), p % 64) if paged else (s, slice(None), p)
                    assert torch.equal(kc[place], ks[at + p - p0]) and torch.equal(vc[place], vs[at + p - p0])
                at += ql
            assert int((kc == 5.0).all(-1).sum()) == kc[..., 0].numel() - G * n      # rows nobody wrote


SHAPES = [(6, 2, 24, 40, 10, 50), (9, 1, 64, 128, 32, 128), (17, 1, 136, 256, 2, 3), (4, 4, 48, 48, 16, 120), (2, 1, 256, 192, 0, 0),
          (16, 4, 128, 256, 0, 0), (3, 1, 8, 96, 6, 400), (1, 1, 16, 8, 32, 64)]


@pytest.mark.parametrize("H, G, dk, dv, rows, largest", SHAPES)
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16, torch.float16])
def test_attention_with_sizes_of_its_own(ops, H, G, dk, dv, rows, largest, dt):
    """Prompts, portions on top of cached rows (pages and blocks) and decode steps with any number of blocks per
    query, with and without distance bias and sink, on tensor cores and with FMA."""
    from yalm_b200.parts.exact_attention import distance_buckets
    rnd = rnd_of(H * 1000 + dk)
    cap, pps, scale = 320, 5, 1.5 * dk ** -0.5
    table = sink = bias_of = None
    if rows:
        rel = 3.0 * rnd(rows, H)                                  # neighbouring buckets differ a lot
        table = dev(rel)[torch.tensor(distance_buckets(rows, largest), device=DEV)].t().contiguous()
        row_of = torch.tensor([distance_bucket(d, rows, largest) for d in range(cap)])
        bias_of = lambda past, T: rel[row_of[(torch.arange(past, past + T)[:, None] - torch.arange(past + T)[None, :]).clamp(min=0)]].permute(2, 0, 1)
        sink = 1.0 + 1.5 * rnd(H)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    for q_lens, past in [([1, 200, 64, 65], [0, 0, 0, 0]), ([3, 64, 1, 70], [100, 200, 311, 63]), ([1, 1, 1, 1], [0, 63, 64, 317])]:
        slots = [2, 0, 3, 1]
        b = B(q_lens, slots)
        n = b.n_tokens
        slot_pos = torch.zeros(4, dtype=torch.int32)
        kc, vc = torch.zeros(4, G, cap, dk, dtype=dt, device=DEV), torch.zeros(4, G, cap, dv, dtype=dt, device=DEV)
        qs, steps, refs = [], [], []
        for ql, p, s in zip(q_lens, past, slots):
            q, k, v = (rnd(ql, H, dk)).to(dt), rnd(p + ql, G, dk).to(dt), rnd(p + ql, G, dv).to(dt)
            slot_pos[s] = p
            rows_in = p + (ql if b.is_decode else 0)              # a decode step's own row is in the cache already
            kc[s, :, :rows_in], vc[s, :, :rows_in] = k[:rows_in].transpose(0, 1).to(DEV), v[:rows_in].transpose(0, 1).to(DEV)
            qs.append(q.reshape(ql, -1))
            steps.append(torch.cat([k[p:].reshape(ql, -1), v[p:].reshape(ql, -1)], 1))
            refs.append(attend(q.double(), k.double(), v.double(), p, scale, bias=bias_of(p, ql) if rows else None, sink=sink))
        ref, q, kv_step, slot_pos = torch.cat(refs), torch.cat(qs).to(DEV), torch.cat(steps).to(DEV).contiguous(), slot_pos.to(DEV)
        pages = torch.randperm(4 * pps + 3, generator=torch.Generator().manual_seed(H))[:4 * pps].reshape(4, pps).to(torch.int32)
        caches = [(kc, vc, None), (paged_copy(kc, pages, pps, dk, dt), paged_copy(vc, pages, pps, dv, dt), pages.to(DEV))]
        for mma in ([True, False] if dt != torch.float32 else [False]):
            for k_cache, v_cache, pt in caches:
                for ns in ((1, 2, 5, 64) if b.is_decode or not mma else (1,)):
                    scratch = {}
                    if ns > 1:
                        scratch = {"part_o": torch.full((n, H, ns, dv), float("nan"), device=DEV),
                                   "part_ml": torch.full((n, H, ns, 2), float("nan"), device=DEV),
                                   "counters": torch.zeros(n * G * -(-(H // G) // 4), dtype=torch.int32, device=DEV)}
                    out = torch.full((n, H * dv), 9.0, dtype=dt, device=DEV)
                    ops.attention_kv(q, kv_step, k_cache, v_cache, b, slot_pos, out, H, G, dk, dv, cap, scale, status, bias=table,
                                     sink=dev(sink) if rows else None, mma=mma, nsplit=ns, pages=pt, **scratch)
                    assert close(out.view(n, H, dv), ref, LOOSE[dt]), (q_lens, mma, pt is not None, ns)
                    if ns > 1:
                        assert int(scratch["counters"].abs().sum()) == 0
    assert int(status) == 0
    # a sequence longer than the caller's bound raises the status instead of reading past anything
    if dt != torch.float32:
        ops.attention_kv(q, kv_step, kc, vc, b, slot_pos, out, H, G, dk, dv, cap, scale, status, mma=True, max_keys=100)
        assert int(status) == ops.ERR_CONTEXT_RANGE


@pytest.mark.parametrize("where", ["prompt", "decode"])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_one_key_at_the_edge_of_a_bucket(ops, where, dt):
    """A key whose score stands far above all others, and a table that forbids one bucket: right inside the
    bucket the key is lost, right outside it takes the whole weight; a sink above every score takes it all."""
    from yalm_b200.parts.exact_attention import distance_buckets
    H, G, dk, dv, n, rows, largest = 2, 1, 16, 24, 200, 16, 120
    edges = distance_buckets(rows, largest)
    rnd = rnd_of(9)
    for bucket in (0, 7, 8, 11, 15):
        lo = edges.index(bucket)
        hi = len(edges) - 1 - edges[::-1].index(bucket)
        rel = torch.zeros(rows, H).double()
        rel[bucket] = -60.0
        table = dev(rel)[torch.tensor(edges, device=DEV)].t().contiguous()
        for back in sorted({d for d in (lo - 1, lo, hi, hi + 1, 150) if 0 <= d < n}):
            loud = n - 1 - back
            q, k, v = 0.05 * rnd(n, H, dk), 0.05 * rnd(n, G, dk), rnd(n, G, dv)
            k[loud], q[:, :, 0] = 0.0, 4.0
            k[loud, :, 0] = 8.0
            q, k, v = q.to(dt), k.to(dt), v.to(dt)
            for sink in (torch.tensor([-3.0, -3.0]).double(), torch.tensor([60.0, -3.0]).double()):
                i = torch.arange(n)
                bias = rel[torch.tensor([distance_bucket(d, rows, largest) for d in range(n)])[(i[:, None] - i[None]).clamp(min=0)]]
                ref = attend(q.double(), k.double(), v.double(), 0, 1.0, bias=bias.permute(2, 0, 1), sink=sink)
                kv = torch.cat([k.reshape(n, -1), v.reshape(n, -1)], 1).to(DEV)
                kc, vc = torch.zeros(1, G, 256, dk, dtype=dt, device=DEV), torch.zeros(1, G, 256, dv, dtype=dt, device=DEV)
                if where == "prompt":
                    b, qq, pos = B([n], [0]), q, 0
                else:
                    b, qq, ref, kv, pos = B([1], [0]), q[n - 1:], ref[n - 1:], kv[n - 1:], n - 1
                    kc[0, :, :n], vc[0, :, :n] = k.transpose(0, 1).to(DEV), v.transpose(0, 1).to(DEV)
                out = torch.empty(qq.shape[0], H * dv, dtype=dt, device=DEV)
                ops.attention_kv(qq.reshape(qq.shape[0], -1).to(DEV), kv.contiguous(), kc, vc, b,
                                 torch.tensor([pos], dtype=torch.int32, device=DEV), out, H, G, dk, dv, 256, 1.0,
                                 torch.zeros(1, dtype=torch.int32, device=DEV), bias=table, sink=dev(sink))
                assert close(out.view(ref.shape), ref, 2e-2 if dt == torch.bfloat16 else 1e-4), (bucket, back, sink.tolist())
                inside = lo <= back <= hi or (bucket == 15 and back >= lo)
                found = (ref[-1, 1] - v[loud, 0].double()).abs().max() < 1e-2
                assert bool(found) == (not inside), (bucket, back)
                if sink[0] > 50:
                    assert out.view(ref.shape)[-1, 0].abs().max() < 1e-3


# heads, key size, value size, rank, tau
GLA_SHAPES = [(3, 20, 36, 12, 8.0), (1, 64, 64, 1, 1.0), (2, 160, 72, 24, 16.0), (3, 10, 13, 3, 4.0), (4, 128, 33, 16, 16.0),
              (2, 256, 40, 70, 2.0), (8, 4, 8, 5, 0.5)]


@pytest.mark.parametrize("H, dk, dv, rank, tau", GLA_SHAPES)
def test_gated_linear_attention(ops, H, dk, dv, rank, tau):
    """Unequal sequences with a carried state; decays from almost 1 to e^-20 per token in one head (runs with
    and without decays of every token); the same in portions and one token at a time; other slots untouched."""
    rnd = rnd_of(H * 100 + dk)
    q_lens, slots = [45, 1, 18, 203, 8], [2, 0, 3, 5, 4]
    b = B(q_lens, slots)
    n = b.n_tokens
    nq, nv = H * dk, H * dv
    cols = (4, 4 + nq, 8 + 2 * nq, 12 + 2 * nq + nv)
    row = cols[3] + rank + 3
    src = rnd(2, n, row)
    w2 = rnd(rank, nq) / rank ** 0.5
    bias = torch.linspace(-6.0, 14.0, nq, dtype=torch.float64)[torch.randperm(nq, generator=torch.Generator().manual_seed(dk))]
    z = src.sum(0)
    q = z[:, cols[0]:cols[0] + nq].view(n, H, dk) * dk ** -0.5
    k, v = z[:, cols[1]:cols[1] + nq].view(n, H, dk), z[:, cols[2]:cols[2] + nv].view(n, H, dv)
    logit = z[:, cols[3]:cols[3] + rank] @ w2 + bias
    logit[60:70] -= 40.0          # a stretch that forgets nearly everything, through one more low-rank value that only it has
    src2 = src.clone()
    src2[:, :, cols[3] + rank:] = 0
    src2[0, 60:70, cols[3] + rank] = -40.0
    w2x = torch.cat([w2, torch.ones(1, nq).double()])
    alpha = torch.exp(F.logsigmoid(logit) / tau).view(n, H, dk)
    S0 = 0.3 * rnd(6, H, dk, dv)
    start = S0.transpose(2, 3).contiguous().float().to(DEV)                     # the library's layout: [H, dv, dk]
    want, last = torch.empty(n, H, dv).double(), {}
    at = 0
    for ql, s in zip(q_lens, slots):
        for h in range(H):
            S = S0[s, h].clone()
            want[at:at + ql, h] = gated_linear(q[at:at + ql, h], k[at:at + ql, h], v[at:at + ql, h], alpha[at:at + ql, h], S)
            last[s, h] = S
        at += ql

    def run(rows, bt, state):
        m = bt.n_tokens
        out = torch.empty(m, nv, device=DEV)
        ops.gla(dev(src2[:, rows]), 2, cols, rank + 1, dev(w2x), dev(bias), tau, torch.full((m, 3 * nq + nv), float("nan"), device=DEV),
                torch.full((m, H), 7, dtype=torch.int32, device=DEV), bt, state, out, H, dk, dv)
        return out

    state = start.clone()
    assert close(run(slice(None), b, state).view(n, H, dv), want, 2e-5)
    for (s, h), S in last.items():
        assert close(state[s, h], S.T, 2e-5), (s, h)
    assert torch.equal(state[1], start[1])
    # the longest sequence in portions, then token by token
    first, s = sum(q_lens[:3]), slots[3]
    for cuts in ([2, 3, 64, 7, 2, 125], [1] * 203):
        state, at, got = start.clone(), first, []
        for c in cuts:
            got.append(run(slice(at, at + c), B([c], [s]), state))
            at += c
        assert close(torch.cat(got).view(-1, H, dv), want[first:first + 203], 2e-5), len(cuts)
        assert close(state[s], torch.stack([last[s, h].T for h in range(H)]), 2e-5)


def test_slow_decays_do_not_drift(ops):
    """Channels that keep a state alive over thousands of tokens: the decays' roundings must not add up."""
    rnd = rnd_of(1)
    H, dk, dv, T = 2, 32, 16, 3000
    src = rnd(1, T, 2 * H * dk + H * dv + 4)
    src[..., -4:] = 0
    bias = torch.linspace(3.0, 12.0, H * dk, dtype=torch.float64)
    cols = (0, H * dk, 2 * H * dk, 2 * H * dk + H * dv)
    q, k = src[0, :, :H * dk].view(T, H, dk) * dk ** -0.5, src[0, :, H * dk:2 * H * dk].view(T, H, dk)
    v = src[0, :, 2 * H * dk:2 * H * dk + H * dv].view(T, H, dv)
    alpha = torch.exp(F.logsigmoid(bias) / 16.0).view(H, dk)
    for cuts in ([T], [700, 1, 2299], [1] * 1500):
        state, got, at = torch.zeros(1, H, dv, dk, device=DEV), [], 0
        for c in cuts:
            out = torch.empty(c, H * dv, device=DEV)
            ops.gla(dev(src[:, at:at + c]), 1, cols, 4, torch.zeros(4, H * dk, device=DEV), dev(bias), 16.0,
                    torch.empty(c, 3 * H * dk + H * dv, device=DEV), torch.empty(c, H, dtype=torch.int32, device=DEV), B([c], [0]),
                    state, out, H, dk, dv)
            got.append(out)
            at += c
        got = torch.cat(got).view(at, H, dv)
        for h in range(H):
            ref = gated_linear(q[:at, h], k[:at, h], v[:at, h], alpha[h].expand(at, dk), torch.zeros(dk, dv).double())
            assert close(got[:, h], ref, 3e-6), (len(cuts), h)


# heads, key size, value size, cap
@pytest.mark.parametrize("H, dk, dv, cap", [(3, 16, 28, 7.0), (1, 64, 64, 1.0), (2, 136, 40, 30.0), (3, 21, 9, 15.0), (4, 128, 31, 15.0),
                                            (2, 256, 64, 15.0), (1, 8, 300, 4.0)])
def test_matrix_memory(ops, H, dk, dv, cap):
    """Gates, maxima and the scan against the plain recurrence: input gates that rise above and fall below the
    running maximum, forget gates of nearly 1 and of nearly 0, a carried state; portions and single tokens."""
    rnd = rnd_of(H * 10 + dk)
    q_lens, slots = [45, 1, 18, 303, 8], [2, 0, 3, 5, 4]
    b = B(q_lens, slots)
    n, nq, nv = b.n_tokens, H * dk, H * dv
    P = -(-(dv + 1) // 4) * 4
    cols = (0, nq, 2 * nq, 2 * nq + nv, 2 * nq + nv + H + 1)
    src = rnd(2, n, cols[4] + H)
    src[0, :, cols[3]:] *= 3.0
    src[0, 90:110, cols[4]:] -= 30.0                              # a stretch that forgets everything
    i_b, f_b = rnd(H) - 1.0, rnd(H) + 4.0
    z = src.sum(0)
    q, k = z[:, :nq].view(n, H, dk) * dk ** -0.5, z[:, nq:2 * nq].view(n, H, dk)
    v = z[:, 2 * nq:2 * nq + nv].view(n, H, dv)
    gi = cap * torch.tanh((z[:, cols[3]:cols[3] + H] + i_b) / cap)
    gf = F.logsigmoid(cap * torch.tanh((z[:, cols[4]:cols[4] + H] + f_b) / cap))
    S0, n0, m0 = 0.3 * rnd(6, H, dk, dv), 0.3 * rnd(6, H, dk), 2.0 * rnd(6, H)
    start = torch.zeros(6, H, P, dk, device=DEV)
    start[:, :, :dv], start[:, :, dv] = dev(S0.transpose(2, 3)), dev(n0)
    # a token's output is a quotient whose denominator may come close to nothing: its pieces are compared, and the
    # output step on the pieces that the kernels themselves made
    want, last, at = torch.empty(n, H, dv + 2).double(), {}, 0
    for ql, s in zip(q_lens, slots):
        for h in range(H):
            S, nn, pieces = S0[s, h].clone(), n0[s, h].clone(), []
            _, m = matrix_memory(q[at:at + ql, h], k[at:at + ql, h], v[at:at + ql, h], gi[at:at + ql, h], gf[at:at + ql, h],
                                 S, nn, float(m0[s, h]), pieces)
            want[at:at + ql, h] = torch.stack(pieces)
            last[s, h] = (S, nn, m)
        at += ql
    gate, w = rnd(2, n, nv + 2), 1.0 + 0.1 * rnd(nv)

    def run(rows, bt, state, maxima):
        m = bt.n_tokens
        act, y = torch.empty(m, H * P + 2 * nq, device=DEV), torch.empty(m, H * P, device=DEV)
        la, put, floor = (torch.empty(m, H, device=DEV) for _ in range(3))
        ops.mlstm_prep(dev(src[:, rows]), 2, cols, dev(i_b), dev(f_b), cap, act, la, put, floor, maxima, bt, H, dk, dv, P)
        ops.ssd_scan(act, None, 0, 0, None, None, None, bt, state, y, H, H, P, dk, steps=(la, put))
        made = y.view(m, H, P).double().cpu()
        o = made[..., :dv] / (torch.maximum(made[..., dv].abs(), floor.double().cpu()) + 1e-6)[..., None]
        final = over_rms(o, 1e-6).reshape(m, nv) * w * torch.sigmoid(gate[:, rows].sum(0)[:, 2:])
        for dt in (torch.float32, torch.bfloat16):
            out = torch.empty(m, nv, dtype=dt, device=DEV)
            ops.gated_heads(y, dev(w), dev(gate[:, rows]), 2, 2, out, H, dv, 1e-6, silu=False, floor=floor)
            assert close(out, final, 1e-5 if dt == torch.float32 else 1e-2)
        return torch.cat([made[..., :dv + 1], floor.double().cpu()[..., None]], -1)

    state, maxima = start.clone(), dev(m0)
    got = run(slice(None), b, state, maxima)
    for part in (slice(0, dv), slice(dv, dv + 1), slice(dv + 1, dv + 2)):
        assert close(got[..., part], want[..., part], 2e-5), part
    for (s, h), (S, nn, m) in last.items():
        assert close(state[s, h, :dv], S.T, 2e-5) and close(state[s, h, dv], nn, 2e-5), (s, h)
        assert abs(float(maxima[s, h]) - m) < 1e-4
    assert torch.equal(state[1], start[1]) and float(state[:, :, dv + 1:].abs().sum()) == 0
    first, s = sum(q_lens[:3]), slots[3]
    for cuts in ([2, 3, 64, 7, 2, 225], [1] * 303):
        state, maxima, at, got = start.clone(), dev(m0), first, []
        for c in cuts:
            got.append(run(slice(at, at + c), B([c], [s]), state, maxima))
            at += c
        got = torch.cat(got)
        for part in (slice(0, dv), slice(dv, dv + 1), slice(dv + 1, dv + 2)):
            assert close(got[..., part], want[first:first + 303, :, part], 2e-5), (len(cuts), part)


# heads, q/k heads, key size, value size
@pytest.mark.parametrize("H, G, dk, dv", [(4, 2, 32, 24), (1, 1, 128, 64), (2, 1, 192, 40), (3, 1, 13, 11), (2, 2, 30, 21), (6, 3, 64, 17),
                                          (4, 1, 256, 8), (3, 3, 8, 4)])
def test_delta_rule_with_one_decay_per_head(ops, H, G, dk, dv):
    """Convolution, unit vectors, betas and decays, then the rule; decays from nearly 1 to e^-40 in one sequence
    (groups that forget too much take every token's own); portions and single tokens; other slots untouched."""
    rnd = rnd_of(H * 10 + dk)
    q_lens, slots = [45, 1, 18, 203, 16], [2, 0, 3, 5, 4]
    b = B(q_lens, slots)
    n, C = b.n_tokens, 2 * G * dk + H * dv
    col_b, col_a = C + 2, C + 2 + H
    src = rnd(2, n, col_a + H + 1)
    src[0, 80:100, col_a:] += 6.0                                 # a stretch that forgets much
    dt_bias, a_log = rnd(H) - 1.0, torch.linspace(-6.0, 2.0, H, dtype=torch.float64)
    z = src.sum(0)
    act0 = F.silu(z[:, :C])
    q, k = unit(act0[:, :G * dk].view(n, G, dk)) * dk ** -0.5, unit(act0[:, G * dk:2 * G * dk].view(n, G, dk))
    v = act0[:, 2 * G * dk:].view(n, H, dv)
    beta = torch.sigmoid(z[:, col_b:col_b + H])
    g = torch.exp(-torch.exp(a_log) * F.softplus(z[:, col_a:col_a + H] + dt_bias))
    S0 = 0.3 * rnd(6, H, dk, dv)
    start = S0.transpose(2, 3).contiguous().float().to(DEV)
    want, last, at = torch.empty(n, H, dv).double(), {}, 0
    for ql, s in zip(q_lens, slots):
        for h in range(H):
            S = S0[s, h].clone()
            hq = h // (H // G)
            want[at:at + ql, h] = delta_rule(q[at:at + ql, hq], k[at:at + ql, hq], v[at:at + ql, h], beta[at:at + ql, h],
                                             g[at:at + ql, h], S)
            last[s, h] = S
        at += ql

    def run(rows, bt, state):
        m = bt.n_tokens
        act = torch.full((m, ops.delta_head_row(H, G, dk, dv)), float("nan"), device=DEV)
        act[:, :C] = dev(act0[rows])
        ops.delta_head_prep(act, dev(src[:, rows]), 2, col_b, col_a, dev(dt_bias), dev(a_log), bt, H, G, dk, dv)
        out = torch.empty(m, H * dv, device=DEV)
        ops.delta_head_scan(act, bt, state, out, H, G, dk, dv)
        return out

    state = start.clone()
    assert close(run(slice(None), b, state).view(n, H, dv), want, 2e-5)
    for (s, h), S in last.items():
        assert close(state[s, h], S.T, 2e-5), (s, h)
    assert torch.equal(state[1], start[1])
    first, s = sum(q_lens[:3]), slots[3]
    for cuts in ([2, 3, 64, 7, 2, 125], [17, 15, 16, 155], [1] * 203):
        state, at, got = start.clone(), first, []
        for c in cuts:
            got.append(run(slice(at, at + c), B([c], [s]), state))
            at += c
        assert close(torch.cat(got).view(-1, H, dv), want[first:first + 203], 2e-5), len(cuts)
        assert close(state[s], torch.stack([last[s, h].T for h in range(H)]), 2e-5)


@pytest.mark.parametrize("heads, size", [(3, 64), (2, 10), (5, 130), (1, 300), (2, 516), (4, 24), (1, 1000), (2, 257)])
def test_gated_heads(ops, heads, size):
    rnd = rnd_of(size)
    for rows in (3, 700):
        y, w, gate = rnd(rows, heads * size), rnd(heads * size), rnd(3, rows, heads * size + 4)
        z = gate.sum(0)[:, 4:]
        for silu in (True, False):
            ref = over_rms(y.view(rows, heads, size), 1e-5).reshape(rows, -1) * w * (F.silu(z) if silu else torch.sigmoid(z))
            for dt in (torch.float32, torch.bfloat16, torch.float16):
                out = torch.empty(rows, heads * size, dtype=dt, device=DEV)
                ops.gated_heads(dev(y), dev(w), dev(gate), 3, 4, out, heads, size, 1e-5, silu=silu)
                assert close(out, ref, {torch.float32: 1e-5, torch.bfloat16: 1e-2, torch.float16: 2e-3}[dt]), (rows, silu, dt)


# ------------------------------------------------------------------ the engine
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_residual_stream_layer_by_layer(name):
    cfg, seed = CONFIGS[name]
    w = weights_of(name)
    toks, _ = steady_tokens(name, 90, seed + 5)
    want = []
    ref = plain_logits(cfg, w, toks, taps=want)
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
        reqs[rid], refs[rid] = steady_tokens(name, n, seed * 10 + k)
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


@pytest.mark.parametrize("kind", ["parallel", "parallel_2"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_needles_in_prompts_portions_and_decoding(dtype, kind):
    cfg, w = needle_model(kind)
    n, at = 420, 100
    last = 39 if kind == "parallel" else 8                 # the distance from which on the far bucket is open again
    if kind == "parallel":
        from yalm_b200.parts.exact_attention import distance_buckets
        last = distance_buckets(16, 40).index(15)
    probes = sorted({at + 1, at + 6, at + 7, at + 8, at + last - 1, at + last, 127, 128, 192, 319, 320, 419})
    toks = needle_tokens(n, [at], probes)
    ref = plain_logits(cfg, w, toks)
    blind = list(toks)
    blind[at] = 9
    lost = plain_logits(cfg, w, blind)
    for p in probes:                                      # a needle lost, or found where the table closes, would show
        back = p - at
        seen = kind == "parallel_2" or back < 8 or back >= last
        assert ((ref[p] - lost[p]).abs().max() > 0.4 * ref[at + 1].abs().max()) == seen, p
    refs, reqs = {"n": ref, "s": ref[:at + last + 3]}, {"n": toks, "s": toks[:at + last + 3]}
    tr = Trace()
    add_whole(tr, {"n": toks})
    add_tail(tr, {"s": reqs["s"]}, tail=last + 4)         # the needle, too, is decoded in some
    add_tail(tr, {"n": toks}, tail=110)
    add_portions(tr, "n", toks, [1, 62, 1, 2, 36, 2, 200])
    lm = _lm(cfg, w, dtype, max_context=512, max_batch=2, max_tokens=tr.max_tokens)
    compare(tr, run_in_process(lm, tr), refs, cfg["vocab"], TOL[dtype])
    # the needle as the sequence's very first token, the probe right after it
    first = needle_tokens(60, [0], [1, 7, 8, 39, 59])
    ref0 = plain_logits(cfg, w, first)
    assert ref0[1].argmax() == NEEDLE
    tr = Trace()
    add_whole(tr, {"f": first})
    add_tail(tr, {"f": first}, tail=59)
    compare(tr, run_in_process(lm, tr), {"f": ref0}, cfg["vocab"], TOL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["tet_a", "tet_b"])
def test_long_decoding_through_the_captured_step(name, dtype):
    cfg, seed = CONFIGS[name]
    w = weights_of(name)
    reqs, refs = {}, {}
    for k, (rid, n) in enumerate({"x": 240, "y": 90, "z": 141}.items()):
        reqs[rid], refs[rid] = steady_tokens(name, n, seed * 7 + k)
    lm = _lm(cfg, w, dtype, max_context=256, max_batch=3)
    forced_decode(lm, reqs, {"x": 30, "y": 3, "z": 65}, refs, TOL[dtype])
    # the same slots again, other requests: nothing of the earlier states is left
    forced_decode(lm, reqs, {"x": 1, "y": 64, "z": 2}, refs, TOL[dtype], order=["z", "x", "y"])


def test_a_request_does_not_depend_on_its_batch():
    cfg, seed = CONFIGS["tet_a"]
    w = weights_of("tet_a")
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
    cfg, seed = CONFIGS["tet_a"]
    w = weights_of("tet_a")
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
    cfg, seed = CONFIGS["tet_c"]
    w = weights_of("tet_c")
    write_model(tmp_path / "model", cfg, w)
    reqs, refs = {}, {}
    for k, (rid, n) in enumerate({"a": 70, "b": 9}.items()):
        reqs[rid], refs[rid] = steady_tokens("tet_c", n, 50 + k)
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
    cfg, _ = CONFIGS["tet_b"]
    with open(tmp_path / "cfg.json", "w") as f:
        json.dump(cfg, f)
    model = str(tmp_path / "model")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, "-m", "yalm_b200", model, "--dtype", "float32", "--random-weights",
                        str(tmp_path / "cfg.json"), "--seed", "3", "--tokens", "5,6,7;9,10", "-n", "6", "-t", "0"],
                       capture_output=True, text=True, cwd=root, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert "Tetodra" in r.stdout
    lines = [l for l in r.stdout.splitlines() if l.startswith("tokens:")]
    w = load_checkpoint(model)
    for line, prompt in zip(lines, ([5, 6, 7], [9, 10])):
        assert [int(t) for t in line.split("(")[0].split()[1:]] == plain_generate_greedy(cfg, w, prompt, 6)
    assert len(lines) == 2
