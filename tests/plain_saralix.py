"""A plain, slow statement of the Saralix decoder in torch on the CPU, one function per mechanism,
written from the design's equations and sharing no code with the library.  It keeps every
sequence's state in a dict so that a prompt can be fed in pieces.

Notation: T tokens of one sequence, width D.  Weights are [out, in] and applied as W x.

    ln(x)             = (x - mean) / sqrt(mean((x - mean)^2) + eps) w
    layer             : x += ln1b(mixer(ln1(x)));  x += ln2b(ff(ln2(x)))
    latent attention  : q = Wq h, per head [dim | rot_dim];  Wdkv h = [c' | kr];  c = c' / rms(c') w_c;
                        qr, kr rotated in halves (YaRN);  key_i = [Wuk_i c | kr],  value_i = Wuv_i c;
                        softmax(scale q.k) over the visible keys, either with a gate sigmoid(Wg h)_i on head
                        i's output, or over a window with exp(sink_i) in the denominator;  Wo
    mamba2            : Win h = [z | x | B | C | dt];  [x | B | C] = silu(conv(.) + b);
                        dt = softplus(dt + dt_bias);  S <- exp(-exp(A) dt) S + dt B x^T;  y = S^T C + D x;
                        g = y silu(z), every norm group over its root mean square, times w;  Wo
    dense             : g = min(Wg h, L), u = clamp(Wu h, L);  Wd (g sigmoid(1.702 g) (u + 1))
    experts           : the `top` largest of z = Wr h, softmax over those;  Wd (silu(Wg h) Wu h)
"""
from __future__ import annotations

import math
from typing import Dict, List

import torch
import torch.nn.functional as F


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def yarn(dims: int, base: float, scaling):
    """Angle per position of each of the dims/2 pairs (float64), and the factor on cos and sin."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=torch.float64), 1.0
    factor, orig = float(scaling["factor"]), float(scaling["original"])

    def dim_of(turns):
        return dims * math.log(orig / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(dim_of(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def rotate_halves(x, positions, freqs, mult):
    """x [T, heads, dims]: the pair (i, i + dims/2) turns by positions[t] * freqs[i], times mult."""
    half = x.shape[-1] // 2
    ang = positions.to(torch.float64)[:, None] * freqs[None, :]
    c, s = (torch.cos(ang) * mult).to(x.dtype)[:, None], (torch.sin(ang) * mult).to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:]
    return torch.cat([u * c - v * s, v * c + u * s], -1)


def visible(n_q: int, past: int, window):
    """bool [n_q, past + n_q]: which keys each of the queries past .. past + n_q - 1 sees."""
    i = torch.arange(past, past + n_q)[:, None]
    j = torch.arange(past + n_q)[None, :]
    ok = j <= i
    return ok if not window else ok & (i - j < window)


def attend(q, k, v, mask, scale, sink=None):
    """q [T, H, d], k [K, H, d], v [K, H, dv]; sink [H] takes part in the denominator alone."""
    s = torch.einsum("thd,khd->htk", q, k) * scale
    s = s.masked_fill(~mask[None], float("-inf"))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink[:, None, None] - top)
    return torch.einsum("htk,khd->thd", e / den, v)


def causal_conv(u, w, bias, before):
    """u [T, C]; w [C, taps], last column the current token's; before [taps - 1, C] the inputs ahead of
    u.  Returns (y, the new ``before``)."""
    taps = w.shape[1]
    full = torch.cat([before, u], 0)
    y = sum(full[j:j + u.shape[0]] * w[:, j] for j in range(taps)) + bias
    return y, full[full.shape[0] - (taps - 1):]


def ssm_scan(x, Bm, Cm, dt, a_log, d_skip, S):
    """One head over T tokens: x [T, P], Bm, Cm [T, N], dt [T]; S [N, P] (changed in place)."""
    out = []
    for t in range(x.shape[0]):
        S.mul_(torch.exp(-torch.exp(a_log) * dt[t]))
        S.add_(dt[t] * torch.outer(Bm[t], x[t]))
        out.append(S.T @ Cm[t] + d_skip * x[t])
    return torch.stack(out)


def clamped_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def route(z, top: int):
    """(chosen experts, weights, margin): the margin is how far the last chosen logit lies above the
    best one left out; a 16-bit computation may rightly decide a close call the other way."""
    order = z.argsort(descending=True)
    chosen = order[:top]
    margin = float(z[order[top - 1]] - z[order[top]]) if top < z.numel() else float("inf")
    return chosen, torch.softmax(z[chosen], -1), margin


class PlainSaralix:
    def __init__(self, config: dict, tensors: Dict[str, torch.Tensor], dtype=torch.float64):
        self.c = config
        self.dt = dtype
        self.w = {k: v.to(dtype) for k, v in tensors.items()}
        self.eps = float(config["norm"]["eps"])
        self.taps = None                                   # called as taps(layer, x [T, D]) after a layer
        self.margins: List[float] = []                     # of every routing decision made, in order

    def new_state(self) -> dict:
        return {"pos": 0, "layers": [dict() for _ in self.c["layers"]]}

    def latent(self, p, m, h, st, pos0, window=None, gated=False, sinks=False):
        w, T = self.w, h.shape[0]
        H, d, rd, dv, rank = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        q = (h @ w[p + "q"].T).view(T, H, d + rd)
        both = h @ w[p + "dkv"].T
        c = over_rms(both[:, :rank], self.eps) * w[p + "dkv.norm"]
        kr = both[:, rank:]
        qr = q[..., d:]
        if rd:
            freqs, mult = yarn(rd, float(m["rot"]["base"]), m["rot"].get("scaling"))
            pos = torch.arange(pos0, pos0 + T)
            qr, kr = rotate_halves(qr, pos, freqs, mult), rotate_halves(kr[:, None], pos, freqs, mult)[:, 0]
        st["c"] = c = torch.cat([st["c"], c]) if "c" in st else c
        st["kr"] = kr = torch.cat([st["kr"], kr]) if "kr" in st else kr
        K = c.shape[0]
        k = torch.cat([(c @ w[p + "uk"].T).view(K, H, d), kr[:, None].expand(K, H, rd)], -1)
        v = (c @ w[p + "uv"].T).view(K, H, dv)
        o = attend(torch.cat([q[..., :d], qr], -1), k, v, visible(T, K - T, window), float(m["scale"]),
                   w[p + "sink"] if sinks else None)
        if gated:
            o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
        return o.reshape(T, H * dv) @ w[p + "o"].T

    def mamba2(self, p, m, h, st):
        w, T = self.w, h.shape[0]
        H, P, N, G = (int(m[k]) for k in ("heads", "vdim", "state", "groups"))
        inner = H * P
        z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], -1)
        if "conv" not in st:
            st["conv"] = torch.zeros(int(m["conv"]) - 1, xbc.shape[1], dtype=h.dtype)
            st["S"] = torch.zeros(H, N, P, dtype=h.dtype)
        xbc, st["conv"] = causal_conv(xbc, w[p + "conv"], w[p + "conv.b"], st["conv"])
        x, Bm, Cm = torch.split(F.silu(xbc), [inner, G * N, G * N], -1)
        x, Bm, Cm = x.view(T, H, P), Bm.view(T, G, N), Cm.view(T, G, N)
        dt = F.softplus(dt + w[p + "dt_bias"])
        y = torch.stack([ssm_scan(x[:, i], Bm[:, i // (H // G)], Cm[:, i // (H // G)], dt[:, i], w[p + "A_log"][i],
                                  w[p + "D"][i], st["S"][i]) for i in range(H)], 1).reshape(T, inner)
        y = y * F.silu(z)
        y = over_rms(y.view(T, int(m["norm_groups"]), -1), self.eps).reshape(T, inner) * w[p + "norm"]
        return y @ w[p + "o"].T

    def experts(self, p, mlp, h):
        w = self.w
        out = torch.zeros_like(h)
        for t in range(h.shape[0]):
            chosen, weights, margin = route(w[p + "router"] @ h[t], int(mlp["router"]["top"]))
            self.margins.append(margin)
            for e, wt in zip(chosen.tolist(), weights):
                g, u = w[f"{p}e{e}.gate"] @ h[t], w[f"{p}e{e}.up"] @ h[t]
                out[t] += wt * (w[f"{p}e{e}.down"] @ (F.silu(g) * u))
        return out

    def forward(self, tokens: List[int], state: dict) -> torch.Tensor:
        """Feeds ``tokens`` as the sequence's next ones; returns logits [T, vocab]."""
        w, eps, pos0 = self.w, self.eps, state["pos"]
        x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
        for i, L in enumerate(self.c["layers"]):
            p, st, m = f"l{i}.", state["layers"][i], L["mixer"]
            h = layer_norm(x, w[p + "norm1"], eps)
            if L["type"] == "latent_attention":
                y = self.latent(p + "mix.", m, h, st, pos0, gated=True)
            elif L["type"] == "latent_attention_2":
                y = self.latent(p + "mix.", m, h, st, pos0, window=int(m["mask"]["size"]), sinks=True)
            elif L["type"] == "mamba2":
                y = self.mamba2(p + "mix.", m, h, st)
            else:
                raise ValueError(L["type"])
            x = x + layer_norm(y, w[p + "norm1b"], eps)
            mlp = L.get("mlp")
            if mlp:
                h = layer_norm(x, w[p + "norm2"], eps)
                if mlp["kind"] == "dense":
                    q = p + "mlp."
                    y = clamped_glu(h @ w[q + "gate"].T, h @ w[q + "up"].T, float(mlp["limit"])) @ w[q + "down"].T
                else:
                    y = self.experts(p + "mlp.", mlp, h)
                x = x + layer_norm(y, w[p + "norm2b"], eps)
            if self.taps is not None:
                self.taps(i, x)
        state["pos"] = pos0 + len(tokens)
        return layer_norm(x, w["final.norm"], eps) @ w["embed"].T
