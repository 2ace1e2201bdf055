"""Shared pieces of the Tetodra tests: small configurations that differ from each other in every size
and option (also values that a model may happen to make equal or 1), random weights by checkpoint
name, references from the plain implementation in 64 bits, and crafted models in which ONE far key
decides a logit."""
from __future__ import annotations

import copy
import functools
from typing import Dict, List

import torch

from plain_tetodra import PlainTetodra


def dense(ff):
    return {"kind": "dense", "ff": ff}


def rotary_layer(heads, kv, dim, vdim, scale, rot, lin, mlp, scales=(0.8, 0.7)):
    """``rot`` = (dims, base) or None; ``lin`` = (heads, dim, vdim, tau, decay rank)."""
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        left["rot"] = {"dims": rot[0], "base": rot[1]}
    right = dict(zip(("heads", "dim", "vdim", "tau", "decay_rank"), lin))
    return {"type": "parallel_2", "mlp": mlp,
            "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}}


def biased_layer(heads, kv, dim, scale, bias, temp, mem, mlp, scales=(0.6, 0.9)):
    """``bias`` = (rows of the table, largest distance); ``temp`` = (coef, every); ``mem`` = (heads, dim, vdim, cap)."""
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale, "bias_rows": bias[0],
            "bias_max": bias[1], "q_temp": {"coef": temp[0], "every": temp[1]}}
    right = dict(zip(("heads", "dim", "vdim", "gate_cap"), mem))
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}}


def delta_layer(heads, kv, dim, vdim, conv, mlp):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def config(vocab, width, layers, eps=1e-5, mult=1.0, scale=1.0):
    return {"architecture": "Tetodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"scale": scale}, "layers": layers}


# every mixer, key and value sizes that differ, a part of a head rotated, a layer without a feed-forward
TET_A = config(211, 64, [
    rotary_layer(6, 2, 24, 40, 0.25, (16, 1e4), (3, 20, 36, 8.0, 12), dense(80)),
    delta_layer(4, 2, 32, 24, 4, dense(48)),
    biased_layer(4, 2, 32, 0.2, (10, 50), (0.25, 16), (3, 16, 28, 7.0), dense(72)),
    rotary_layer(4, 4, 16, 48, 0.3, (16, 500.0), (2, 36, 20, 16.0, 5), None)], mult=0.8, scale=3.0)
# more query heads per key head than a tile of the decode attention holds, no rotation, strong decays (tau 1),
# and everything that can be 1: one head, one key head, constants of 1
TET_B = config(300, 96, [
    rotary_layer(9, 1, 64, 128, 0.125, None, (1, 64, 64, 1.0, 1), dense(64), (1.0, 1.0)),
    biased_layer(1, 1, 64, 0.03, (32, 128), (1.0, 1), (1, 64, 64, 1.0), dense(120), (1.0, 1.0)),
    delta_layer(1, 1, 128, 64, 2, dense(56))], eps=1e-6)
# a width that is no multiple of 8 (products on the FMA kernel), sizes that are no multiple of 4 or 8 (no
# 16-byte pieces anywhere), a table of two rows
TET_C = config(130, 100, [
    delta_layer(3, 1, 13, 11, 8, dense(50)),
    biased_layer(5, 5, 10, 0.3, (2, 7), (0.4, 7.5), (3, 21, 9, 15.0), dense(30)),
    rotary_layer(6, 3, 14, 9, 0.25, (6, 100.0), (3, 10, 13, 4.0, 3), dense(36)),
    delta_layer(2, 2, 30, 21, 3, None)], mult=0.6, scale=2.5)
# keys and values of more than 128, queries of 17 heads over one key head, states of more than 128 rows
TET_D = config(150, 72, [
    rotary_layer(17, 1, 136, 256, 0.08, (136, 1e6), (2, 160, 72, 16.0, 24), dense(40)),
    biased_layer(2, 1, 200, 0.07, (16, 20), (0.1, 100), (2, 136, 40, 30.0), None),
    delta_layer(2, 1, 192, 40, 5, dense(64))], mult=0.9, scale=4.0)
CONFIGS = {"tet_a": (TET_A, 11), "tet_b": (TET_B, 22), "tet_c": (TET_C, 33), "tet_d": (TET_D, 44)}

# Largest logit error relative to the request's largest logit.
TOL = {"float32": 1e-4, "bfloat16": 6e-2, "float16": 8e-3}


def make_weights(cfg: dict, seed: int, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    mat = lambda r, c, std: (std * torch.randn(r, c, generator=g)).to(dtype)
    vec = lambda n, std, mean=0.0: (mean + std * torch.randn(n, generator=g)).to(dtype)
    conv = lambda c, taps: (0.4 * torch.randn(c, taps, generator=g) + torch.eye(taps)[-1]).to(dtype)
    a = D ** -0.5
    w = {"embed": mat(V, D, 0.7 / cfg["embedding"]["scale"] ** 0.5), "final.norm": vec(D, 0.1, 1.0)}
    for i, L in enumerate(cfg["layers"]):
        p, m, q = f"l{i}", L["mixer"], f"l{i}.mix"
        w[f"{p}.norm1"], w[f"{p}.ls1"] = vec(D, 0.1, 1.0), vec(D, 0.3, 0.8)
        if L["type"] == "delta":
            H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for x, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                w[f"{q}.{x}"], w[f"{q}.{x}.conv"] = mat(rows, D, 1.5 * a), conv(rows, taps)
            w[f"{q}.b"], w[f"{q}.a"] = mat(H, D, 1.5 * a), mat(H, D, a)
            # decays from nearly 1 (a state that remembers hundreds of tokens) down to a few tokens
            w[f"{q}.A_log"], w[f"{q}.dt_bias"] = (-5.0 + 6.0 * torch.rand(H, generator=g)).to(dtype), vec(H, 1.0, -1.0)
            w[f"{q}.g"], w[f"{q}.norm"], w[f"{q}.o"] = mat(H * dv, D, 1.5 * a), vec(dv, 0.1, 1.0), mat(D, H * dv, (H * dv) ** -0.5)
        else:
            l, r = m["left"], m["right"]
            H, G, d, dv = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            w[f"{q}.left.q"], w[f"{q}.left.k"] = mat(H * d, D, 1.5 * a), mat(G * d, D, 1.5 * a)
            w[f"{q}.left.o"] = mat(D, H * dv, (H * dv) ** -0.5)
            H2, d2, dv2 = r["heads"], r["dim"], r["vdim"]
            for x, rows in (("q", H2 * d2), ("k", H2 * d2), ("v", H2 * dv2), ("g", H2 * dv2)):
                w[f"{q}.right.{x}"] = mat(rows, D, 1.2 * a)
            w[f"{q}.right.o"] = mat(D, H2 * dv2, (H2 * dv2) ** -0.5)
            if L["type"] == "parallel":
                w[f"{q}.left.q.norm"], w[f"{q}.left.k.norm"] = vec(d, 0.2, 1.0), vec(d, 0.2, 1.0)
                w[f"{q}.left.rel"], w[f"{q}.left.sink"] = mat(l["bias_rows"], H, 1.5), vec(H, 1.5, 1.0)
                w[f"{q}.right.norm"] = vec(H2 * dv2, 0.1, 1.0)
                # forget gates from nearly 1 down, input gates on both sides of the running maximum
                w[f"{q}.right.i"], w[f"{q}.right.i.b"] = mat(H2, D, 2.0 * a), vec(H2, 1.0, -1.0)
                w[f"{q}.right.f"], w[f"{q}.right.f.b"] = mat(H2, D, a), vec(H2, 1.5, 4.0)
            else:
                w[f"{q}.left.v"] = mat(G * dv, D, a)
                w[f"{q}.right.norm"] = vec(dv2, 0.1, 1.0)
                rank = r["decay_rank"]
                w[f"{q}.right.a1"], w[f"{q}.right.a2"] = mat(rank, D, 1.5 * a), mat(H2 * d2, rank, rank ** -0.5)
                w[f"{q}.right.a2.b"] = vec(H2 * d2, 2.0, 1.0)
        if L["mlp"]:
            ff = L["mlp"]["ff"]
            w[f"{p}.ls2"] = vec(D, 0.3, 0.7)
            w[f"{p}.mlp.gate"], w[f"{p}.mlp.up"] = mat(ff, D, 1.5 * a), mat(ff, D, 1.5 * a)
            w[f"{p}.mlp.down"] = mat(D, ff, ff ** -0.5)
    return w


def weights_of(name: str, dtype=torch.bfloat16):
    cfg, seed = CONFIGS[name]
    return make_weights(cfg, seed, dtype)


def random_tokens(n: int, vocab: int, seed: int) -> List[int]:
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def plain_logits(cfg, w, toks, pieces=None, taps=None):
    """Logits [len(toks), vocab] of the plain implementation in 64 bits, the prompt fed whole or in the
    given pieces."""
    m = PlainTetodra(cfg, w, torch.float64)
    m.taps = taps
    st = m.new_state()
    out, at = [], 0
    for n in (pieces or [len(toks)]):
        out.append(m.forward(toks[at:at + n], st))
        at += n
    if at < len(toks):
        out.append(m.forward(toks[at:], st))
    return torch.cat(out).float()


@functools.lru_cache(maxsize=None)
def steady_tokens(name: str, n: int, seed: int):
    """n random tokens for a configuration of ``CONFIGS`` and their reference logits, drawn one after the other so
    that the plain model's own logits stay near when every weight moves by one rounding of the 16-bit type.  (The
    norms behind the recurrences blow up what is nearly nothing -- a first key across from its query -- and
    then no 16-bit run can be held to a bound.)"""
    cfg, w = CONFIGS[name][0], weights_of(name)
    g = torch.Generator().manual_seed(seed)
    moved = {k: v.double() * (1.0 + 2.0 ** -9 * torch.randn(v.shape, generator=g)) for k, v in w.items()}
    a, b = PlainTetodra(cfg, w), PlainTetodra(cfg, moved)
    sa, sb = a.new_state(), b.new_state()
    toks, rows = [], []
    for _ in range(n):
        best = None
        for _ in range(40):
            t = int(torch.randint(0, cfg["vocab"], (1,), generator=g))
            ta, tb = copy.deepcopy(sa), copy.deepcopy(sb)
            row = a.forward([t], ta)[0]
            err = float((b.forward([t], tb)[0] - row).abs().max() / row.abs().max())
            if best is None or err < best[0]:
                best = (err, t, row, ta, tb)
            if err < 0.3 * TOL["bfloat16"]:
                break
        _, t, row, sa, sb = best
        toks.append(t)
        rows.append(row)
    return toks, torch.stack(rows).float()


def plain_generate_greedy(cfg, w, prompt: List[int], n_new: int) -> List[int]:
    m = PlainTetodra(cfg, w, torch.float64)
    st = m.new_state()
    logits = m.forward(list(prompt), st)
    out = []
    for _ in range(n_new):
        out.append(int(logits[-1].argmax()))
        logits = m.forward([out[-1]], st)
    return out


def add_portions(tr, rid: str, toks: List[int], sizes: List[int], tag="p"):
    """One request whose prompt comes in portions of the given sizes (the last takes the rest),
    logits at every position."""
    name, at = f"{tag}-{rid}", 0
    tr.need([len(toks)])
    cuts = list(sizes)
    while at < len(toks):
        n = min(cuts.pop(0) if cuts else len(toks), len(toks) - at)
        last = at + n == len(toks)
        tr.add([{"id": name, "tokens": toks[at:at + n], "want": list(range(n))}], [name] if last else [],
               [(rid, p) for p in range(at, at + n)])
        at += n


# ---------------------------------------------------------------------------
# One layer whose attention makes ONE key stand out: the keys of the token NEEDLE alone lie along a direction
# that only the token PROBE asks for.  Whether a probe finds the needle -- hundreds of positions back, at a
# page's border, at the edge of a distance bucket -- decides feature 0 of the layer's output, and with it the
# probe's logits.  The recurrent branch writes nothing.
NEEDLE, PROBE = 3, 5


def needle_model(kind: str, heads=3, dim=32, width=48, vocab=40):
    """``kind``: "parallel" (keys are values; the table is low everywhere but in the buckets it has for distances
    below 8 and from 40 on) or "parallel_2"."""
    g = torch.Generator().manual_seed(17)
    rnd = lambda *shape: 0.05 * torch.randn(*shape, generator=g)
    E = 0.3 * torch.randn(vocab, width, generator=g)
    E[:, :2] = 0
    E[:, 2:] -= E[:, 2:].mean(-1, keepdim=True)          # the layer norm then leaves features 0 and 1 of the others at zero
    E[NEEDLE], E[PROBE] = 0, 0
    E[NEEDLE, 0], E[PROBE, 1] = 2.0, 2.0
    mem = (1, 8, 8, 5.0) if kind == "parallel" else (1, 8, 8, 8.0, 4)
    if kind == "parallel":
        layer = biased_layer(heads, 1, dim, 0.7, (16, 40), (0.05, 100), mem, None, (1.0, 1.0))
    else:
        layer = rotary_layer(heads, 1, dim, dim, 0.7, None, mem, None, (1.0, 1.0))
    cfg = config(vocab, width, [layer])
    w = {k: v.float() for k, v in make_weights(cfg, 5).items()}
    q, k, o = rnd(heads * dim, width), rnd(dim, width), 0.05 * torch.randn(width, heads * dim, generator=g)
    k[0] = 0
    k[0, 0] = 4.0
    q[:, 1] = 0
    for h in range(heads):
        q[h * dim] = 0
        q[h * dim, 1] = 4.0
        o[0, h * dim] = 1.0
    w.update({"embed": E, "final.norm": torch.ones(width), "l0.norm1": torch.ones(width), "l0.ls1": torch.ones(width),
              "l0.mix.left.q": q, "l0.mix.left.k": k, "l0.mix.left.o": o, "l0.mix.right.o": torch.zeros_like(w["l0.mix.right.o"])})
    if kind == "parallel":
        w["l0.mix.left.q.norm"], w["l0.mix.left.k.norm"] = torch.ones(dim), torch.ones(dim)
        rel = torch.full((16, heads), -30.0)
        rel[:8], rel[15] = 0.0, 0.0                      # distances 0 .. 7 and those of the last bucket
        w["l0.mix.left.rel"] = rel + 0.1 * torch.randn(16, heads, generator=g)
        w["l0.mix.left.sink"] = torch.full((heads,), -2.0)
    else:
        v = rnd(dim, width)
        v[0] = 0
        v[0, 0] = 2.0
        w["l0.mix.left.v"] = v
    return cfg, {key: v.to(torch.bfloat16) for key, v in w.items()}


def needle_tokens(n: int, needles: List[int], probes: List[int], vocab=40, seed=0) -> List[int]:
    g = torch.Generator().manual_seed(seed)
    toks = torch.randint(8, vocab, (n,), generator=g).tolist()
    for p in needles:
        toks[p] = NEEDLE
    for p in probes:
        toks[p] = PROBE
    return toks
