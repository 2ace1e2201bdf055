"""Shared pieces of the Saralix tests: small configurations that differ from each other in every size
and option (also values that a model may happen to make equal or 1), random weights by checkpoint
name, references from the plain implementation in 64 bits, and a crafted model in which ONE far key
decides a logit."""
from __future__ import annotations

import copy
from typing import Dict, List

import torch

from plain_saralix import PlainSaralix


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def yarn_scaling(factor, original, fast=32.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def latent_layer(heads, dim, rot_dim, vdim, rank, scale, base, mlp, scaling=None, window=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if scaling:
        m["rot"]["scaling"] = scaling
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention_2" if window else "latent_attention", "mixer": m, "mlp": mlp}


def mamba_layer(heads, vdim, state, groups, conv, norm_groups, mlp):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}, "mlp": mlp}


# every mixer and feed-forward, key and value sizes that differ, a layer without a feed-forward
SARA_A = {
    "architecture": "Saralix", "vocab": 211, "width": 64, "norm": {"eps": 1e-5},
    "layers": [latent_layer(3, 24, 8, 16, 40, 0.2, 1e4, dense(80, 1.5), yarn_scaling(4.0, 64), window=33),
               mamba_layer(6, 20, 16, 3, 3, 2, moe(6, 2, 40)),
               latent_layer(2, 16, 16, 32, 56, 0.25, 5e4, None, yarn_scaling(16.0, 128, 8.0, 2.0)),
               mamba_layer(4, 24, 40, 1, 2, 4, dense(48, 7.0))],
}
# more heads than one tile of the tensor-core attention holds, a window of one page, everything that can be
# 1: one head, one group, one norm group, one expert per token; rotation without scaling
SARA_B = {
    "architecture": "Saralix", "vocab": 300, "width": 96, "norm": {"eps": 1e-6},
    "layers": [latent_layer(18, 8, 16, 24, 72, 0.3, 1e4, moe(3, 1, 56)),
               mamba_layer(1, 64, 128, 1, 5, 1, dense(64, 0.5)),
               latent_layer(1, 48, 24, 64, 200, 0.15, 2e5, moe(4, 4, 32), yarn_scaling(2.0, 1024), window=64)],
}
# a width that is no multiple of 8 (products on the FMA kernel), sizes that are no multiple of 4 or 8 (no
# 16-byte pieces anywhere), a window shorter than any prompt, one rotated pair
SARA_C = {
    "architecture": "Saralix", "vocab": 130, "width": 100, "norm": {"eps": 1e-5},
    "layers": [mamba_layer(3, 10, 21, 3, 8, 5, dense(50, 2.5)),
               latent_layer(5, 10, 2, 12, 21, 0.3, 100.0, moe(5, 2, 30), window=7),
               latent_layer(2, 14, 6, 9, 30, 0.2, 1e4, dense(36, 3.0), yarn_scaling(3.0, 50))],
}
# a latent row wider than 256 features under a window of one position, then a causal one
SARA_D = {
    "architecture": "Saralix", "vocab": 150, "width": 72, "norm": {"eps": 1e-5},
    "layers": [latent_layer(4, 32, 16, 40, 300, 0.15, 1e4, None, window=1),
               latent_layer(3, 16, 32, 136, 288, 0.2, 1e6, dense(40, 4.0), yarn_scaling(8.0, 256))],
}
CONFIGS = {"sara_a": (SARA_A, 11), "sara_b": (SARA_B, 22), "sara_c": (SARA_C, 33), "sara_d": (SARA_D, 44)}

# Largest logit error relative to the request's largest logit.
TOL = {"float32": 1e-4, "bfloat16": 6e-2, "float16": 8e-3}
# a routing decision closer than this (in logits) may fall the other way in 16 bits
CLOSE_CALL = 0.1


def make_weights(cfg: dict, seed: int, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    mat = lambda r, c, std: (std * torch.randn(r, c, generator=g)).to(dtype)
    vec = lambda n, std, mean=0.0: (mean + std * torch.randn(n, generator=g)).to(dtype)
    a = D ** -0.5
    w = {"embed": mat(V, D, 0.7), "final.norm": vec(D, 0.1, 1.0)}
    for i, L in enumerate(cfg["layers"]):
        p, m, q = f"l{i}", L["mixer"], f"l{i}.mix"
        w[f"{p}.norm1"], w[f"{p}.norm1b"] = vec(D, 0.1, 1.0), vec(D, 0.05, 0.5)
        if L["type"] == "mamba2":
            H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            inner, C = H * P, H * P + 2 * G * N
            w[f"{q}.in"] = mat(inner + C + H, D, 1.5 * a)
            w[f"{q}.conv"] = (0.4 * torch.randn(C, m["conv"], generator=g) + torch.eye(m["conv"])[-1]).to(dtype)
            w[f"{q}.conv.b"] = vec(C, 0.2)
            # decays from nearly 1 (a state that remembers hundreds of tokens) down to a few tokens
            w[f"{q}.A_log"] = (-5.0 + 6.0 * torch.rand(H, generator=g)).to(dtype)
            w[f"{q}.dt_bias"], w[f"{q}.D"] = vec(H, 1.0, -1.0), vec(H, 0.3, 1.0)
            w[f"{q}.norm"], w[f"{q}.o"] = vec(inner, 0.1, 1.0), mat(D, inner, inner ** -0.5)
        else:
            H, d, rd, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w[f"{q}.q"], w[f"{q}.dkv"] = mat(H * (d + rd), D, 1.5 * a), mat(rank + rd, D, 1.5 * a)
            w[f"{q}.dkv.norm"] = vec(rank, 0.1, 1.0)
            w[f"{q}.uk"], w[f"{q}.uv"] = mat(H * d, rank, 1.5 * rank ** -0.5), mat(H * dv, rank, rank ** -0.5)
            w[f"{q}.o"] = mat(D, H * dv, (H * dv) ** -0.5)
            if L["type"] == "latent_attention":
                w[f"{q}.g"] = mat(H, D, 2.0 * a)
            else:
                w[f"{q}.sink"] = vec(H, 1.5, 1.0)            # of the scores' own size, unequal over the heads
        mlp = L["mlp"]
        if mlp:
            w[f"{p}.norm2"], w[f"{p}.norm2b"] = vec(D, 0.1, 1.0), vec(D, 0.05, 0.5)
            glu = lambda n, ff: {f"{n}.gate": mat(ff, D, 1.5 * a), f"{n}.up": mat(ff, D, 1.5 * a),
                                 f"{n}.down": mat(D, ff, ff ** -0.5)}
            if mlp["kind"] == "dense":
                w.update(glu(f"{p}.mlp", mlp["ff"]))
            else:
                w[f"{p}.mlp.router"] = mat(mlp["router"]["experts"], D, 3.0 * a)
                for j in range(mlp["router"]["experts"]):
                    w.update(glu(f"{p}.mlp.e{j}", mlp["expert"]["ff"]))
    return w


def weights_of(name: str, dtype=torch.bfloat16):
    cfg, seed = CONFIGS[name]
    return make_weights(cfg, seed, dtype)


def random_tokens(n: int, vocab: int, seed: int) -> List[int]:
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def plain_logits(cfg, w, toks, pieces=None, taps=None):
    """(logits [len(toks), vocab] of the plain implementation in 64 bits, the prompt fed whole or in the
    given pieces; the implementation, which remembers its routing margins)."""
    m = PlainSaralix(cfg, w, torch.float64)
    m.taps = taps
    st = m.new_state()
    out, at = [], 0
    for n in (pieces or [len(toks)]):
        out.append(m.forward(toks[at:at + n], st))
        at += n
    if at < len(toks):
        out.append(m.forward(toks[at:], st))
    return torch.cat(out).float(), m


def safe_tokens(cfg, w, n: int, seed: int):
    """n random tokens, drawn one after the other so that no routing decision of the plain
    implementation is a close call (a token that brings one is drawn again), and their reference logits."""
    g = torch.Generator().manual_seed(seed)
    m = PlainSaralix(cfg, w, torch.float64)
    st = m.new_state()
    toks, rows = [], []
    while len(toks) < n:
        for _ in range(200):
            t = int(torch.randint(0, cfg["vocab"], (1,), generator=g))
            trial = copy.deepcopy(st)
            m.margins = []
            row = m.forward([t], trial)
            if not m.margins or min(m.margins) >= CLOSE_CALL:
                break
        else:
            raise AssertionError("no token without a close routing call was found")
        st = trial
        toks.append(t)
        rows.append(row[0])
    return toks, torch.stack(rows).float()


def plain_generate_greedy(cfg, w, prompt: List[int], n_new: int) -> List[int]:
    m = PlainSaralix(cfg, w, torch.float64)
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
# One latent layer whose attention makes ONE key stand out: the token NEEDLE alone fills the latent's first
# feature, which every head's unrotated key and value read, and only the token PROBE asks along it.
# Whether a probe finds the needle -- hundreds of positions back, at a page's border, just inside or just
# outside a window -- decides feature 0 of the layer's (normed) output, and with it the probe's logits.
NEEDLE, PROBE = 3, 5


def needle_model(window=None, heads=3, dim=16, rd=8, vdim=24, rank=40, width=48, vocab=40, scale=0.5, sink=1.0):
    g = torch.Generator().manual_seed(17 + (window or 0))
    bf = torch.bfloat16
    rnd = lambda *shape: 0.05 * torch.randn(*shape, generator=g)
    E = 0.3 * torch.randn(vocab, width, generator=g)
    E[:, :2] = 0
    E[:, 2:] -= E[:, 2:].mean(-1, keepdim=True)          # the layer norm then leaves feature 0 of the others at zero
    E[NEEDLE], E[PROBE] = 0, 0
    E[NEEDLE, 0], E[PROBE, 1] = 2.0, 2.0
    q, dkv, uk, uv = rnd(heads * (dim + rd), width), rnd(rank + rd, width), rnd(heads * dim, rank), rnd(heads * vdim, rank)
    o = 0.05 * torch.randn(width, heads * vdim, generator=g)
    dkv[0] = 0
    dkv[0, 0] = 4.0
    for h in range(heads):
        q[h * (dim + rd)] = 0
        q[h * (dim + rd), 1] = 2.0
        uk[h * dim], uv[h * vdim] = 0, 0
        uk[h * dim, 0] = 1.0
        uv[h * vdim, 0] = 2.0
        o[0, h * vdim] = 2.0
    w = {"embed": E, "final.norm": torch.ones(width), "l0.norm1": torch.ones(width), "l0.norm1b": torch.ones(width),
         "l0.mix.q": q, "l0.mix.dkv": dkv, "l0.mix.dkv.norm": torch.ones(rank), "l0.mix.uk": uk, "l0.mix.uv": uv, "l0.mix.o": o}
    if window:
        w["l0.mix.sink"] = sink * torch.ones(heads) + 0.5 * torch.randn(heads, generator=g)
    else:
        w["l0.mix.g"] = rnd(heads, width)
    cfg = {"architecture": "Saralix", "vocab": vocab, "width": width, "norm": {"eps": 1e-5},
           "layers": [latent_layer(heads, dim, rd, vdim, rank, scale, 1e4, None, yarn_scaling(4.0, 64), window=window)]}
    return cfg, {k: v.to(bf) for k, v in w.items()}


def needle_tokens(n: int, needles: List[int], probes: List[int], vocab=40, seed=0) -> List[int]:
    g = torch.Generator().manual_seed(seed)
    toks = torch.randint(8, vocab, (n,), generator=g).tolist()
    for p in needles:
        toks[p] = NEEDLE
    for p in probes:
        toks[p] = PROBE
    return toks
