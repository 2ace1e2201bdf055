"""A plain, slow statement of the Tetodra decoder in torch on the CPU, one function per mechanism,
written from the design's equations and sharing no code with the library.  It keeps every
sequence's state in a dict so that a prompt can be fed in pieces.

Notation: T tokens of one sequence, width D.  Weights are [out, in] and applied as W x.

    ln(x)        = (x - mean) / sqrt(mean((x - mean)^2) + eps) w
    layer        : h = ln1(x);  x += r (mixer(h) ls1 + ff(h) ls2)
    parallel     : a (biased attention) + b (matrix memory), both on h
    parallel_2   : a (rotary attention) + b (gated linear attention), both on h
    biased       : q = Wq h, k = v = Wk h;  q, k over their rms per head times a weight;
                   q *= 1 + c ln(floor((p + 1) / e) + 1);  score = s q.k + table[bucket(i - j), head];
                   causal, exp(sink_head) in the denominator;  Wo
    rotary       : q, k, v;  the first `dims` of q, k turned in halves;  causal softmax(s q.k) v;  Wo
    matrix memory: i = cap tanh((Wi h + b) / cap), f = logsigmoid(cap tanh((Wf h + b) / cap)),
                   m' = max(f + m, i);  S <- e^(f + m - m') S + e^(i - m') k v^T, n likewise with k;
                   o = S^T q / (max(|n.q|, e^-m') + 1e-6);  over its rms, times w, times sigmoid(Wg h);  Wo
    linear       : S <- diag(sigmoid(z)^(1/tau)) S + k v^T, o = S^T q, z = Wa2 Wa1 h + b;
                   o over its rms times w, times silu(Wg h);  Wo
    delta        : q, k, v = silu(conv(W. h)), q and k unit vectors, q / sqrt(dim);  beta = sigmoid(Wb h);
                   g = exp(-exp(A) softplus(Wa h + dt));  S <- g S;  u = beta (v - S^T k);  S += k u^T;
                   o = S^T q, over its rms times w, times silu(Wg h);  Wo
    ff           : Wd (silu(Wg h) Wu h)
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


def rotate_halves(x, positions, dims: int, base: float):
    """x [T, heads, size]: the pair (i, i + dims/2) of the first ``dims`` features turns by
    positions[t] * base^(-2i/dims)."""
    if not dims:
        return x
    half = dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def distance_bucket(n: int, rows: int, largest: int) -> int:
    """The bias table's row for a key n positions back: one row per distance for the nearest half of
    the rows, logarithmically wider ones up to the distance ``largest``, the last row for all beyond."""
    half = rows // 2
    if n < half:
        return n
    where = math.log(n / half) / math.log(largest / half) * (rows - half)
    near = round(where)
    step = near if abs(where - near) < 1e-9 else math.floor(where)      # an edge is an edge, however log rounds
    return min(rows - 1, half + step)


def query_temperature(p: int, coef: float, every: float) -> float:
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1)


def attend(q, k, v, past: int, scale: float, bias=None, sink=None):
    """q [T, H, d] at positions past .., k [K, G, d], v [K, G, dv] from position 0; head h reads key
    head h // (H / G).  bias [H, T, K] joins the scaled scores; sink [H] the denominator alone."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    k, v = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
    s = torch.einsum("thd,khd->htk", q, k) * scale
    if bias is not None:
        s = s + bias
    i = torch.arange(past, past + T)[:, None]
    j = torch.arange(k.shape[0])[None, :]
    s = s.masked_fill((j > i)[None], float("-inf"))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink[:, None, None] - top)
    return torch.einsum("htk,khd->thd", e / den, v)


def matrix_memory(q, k, v, i, f, S, n, m: float, pieces=None):
    """One head over T tokens: q, k [T, dk], v [T, dv], i, f [T] (logarithms); S [dk, dv], n [dk] changed in
    place.  Returns (o [T, dv], the new m); ``pieces``, a list, receives every token's S^T q, n.q and e^-m."""
    out = []
    for t in range(q.shape[0]):
        mt = max(float(f[t]) + m, float(i[t]))
        keep, put = math.exp(float(f[t]) + m - mt), math.exp(float(i[t]) - mt)
        S.mul_(keep).add_(put * torch.outer(k[t], v[t]))
        n.mul_(keep).add_(put * k[t])
        out.append(S.T @ q[t] / (max(abs(float(n @ q[t])), math.exp(-mt)) + 1e-6))
        if pieces is not None:
            pieces.append(torch.cat([S.T @ q[t], torch.stack([n @ q[t], q.new_tensor(math.exp(-mt))])]))
        m = mt
    return torch.stack(out), m


def gated_linear(q, k, v, alpha, S):
    """One head over T tokens: q, k, alpha [T, dk], v [T, dv]; S [dk, dv] changed in place."""
    out = []
    for t in range(q.shape[0]):
        S.mul_(alpha[t][:, None]).add_(torch.outer(k[t], v[t]))
        out.append(S.T @ q[t])
    return torch.stack(out)


def delta_rule(q, k, v, beta, g, S):
    """One head over T tokens: q, k [T, dk], v [T, dv], beta, g [T]; S [dk, dv] changed in place."""
    out = []
    for t in range(q.shape[0]):
        S.mul_(g[t])
        u = beta[t] * (v[t] - S.T @ k[t])
        S.add_(torch.outer(k[t], u))
        out.append(S.T @ q[t])
    return torch.stack(out)


def causal_conv(u, w, before):
    """u [T, C]; w [C, taps], last column the current token's; before [taps - 1, C] the inputs ahead of
    u.  Returns (y, the new ``before``)."""
    taps = w.shape[1]
    full = torch.cat([before, u], 0)
    return sum(full[j:j + u.shape[0]] * w[:, j] for j in range(taps)), full[full.shape[0] - (taps - 1):]


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


class PlainTetodra:
    def __init__(self, cfg: dict, weights: Dict[str, torch.Tensor], dtype=torch.float64):
        self.cfg = cfg
        self.dtype = dtype
        self.w = {k: v.to(dtype) for k, v in weights.items()}
        self.eps = cfg["norm"]["eps"]
        self.taps = None                # a list that receives the residual stream after every layer

    def new_state(self) -> dict:
        return {"pos": 0, "layers": [{} for _ in self.cfg["layers"]]}

    # ---- mixers: h [T, D] at positions st["pos"] .. ----
    def keys_so_far(self, st, name, new):
        old = st.get(name)
        st[name] = new if old is None else torch.cat([old, new], 0)
        return st[name]

    def biased_attention(self, p, m, h, past, st):
        w, T = self.w, h.shape[0]
        H, G, d = m["heads"], m["kv_heads"], m["dim"]
        q = (h @ w[f"{p}.q"].T).view(T, H, d)
        raw = (h @ w[f"{p}.k"].T).view(T, G, d)
        q = over_rms(q, self.eps) * w[f"{p}.q.norm"]
        k = over_rms(raw, self.eps) * w[f"{p}.k.norm"]
        temp = [query_temperature(past + t, m["q_temp"]["coef"], m["q_temp"]["every"]) for t in range(T)]
        q = q * torch.tensor(temp, dtype=self.dtype)[:, None, None]
        K, V = self.keys_so_far(st, "k", k), self.keys_so_far(st, "v", raw)
        table = w[f"{p}.rel"]
        row = torch.tensor([distance_bucket(n, table.shape[0], m["bias_max"]) for n in range(K.shape[0])])
        back = (torch.arange(past, past + T)[:, None] - torch.arange(K.shape[0])[None, :]).clamp(min=0)
        o = attend(q, K, V, past, m["scale"], bias=table[row[back]].permute(2, 0, 1), sink=w[f"{p}.sink"])
        return o.reshape(T, -1) @ w[f"{p}.o"].T

    def rotary_attention(self, p, m, h, past, st):
        w, T = self.w, h.shape[0]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        pos = torch.arange(past, past + T)
        rot = m.get("rot") or {"dims": 0, "base": 1.0}
        q = rotate_halves((h @ w[f"{p}.q"].T).view(T, H, d), pos, rot["dims"], rot["base"])
        k = rotate_halves((h @ w[f"{p}.k"].T).view(T, G, d), pos, rot["dims"], rot["base"])
        K, V = self.keys_so_far(st, "k", k), self.keys_so_far(st, "v", (h @ w[f"{p}.v"].T).view(T, G, dv))
        return attend(q, K, V, past, m["scale"]).reshape(T, -1) @ w[f"{p}.o"].T

    def memory(self, p, m, h, st):
        w, T = self.w, h.shape[0]
        H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
        q = (h @ w[f"{p}.q"].T).view(T, H, d) * d ** -0.5
        k, v = (h @ w[f"{p}.k"].T).view(T, H, d), (h @ w[f"{p}.v"].T).view(T, H, dv)
        i = cap * torch.tanh((h @ w[f"{p}.i"].T + w[f"{p}.i.b"]) / cap)
        f = F.logsigmoid(cap * torch.tanh((h @ w[f"{p}.f"].T + w[f"{p}.f.b"]) / cap))
        if "S" not in st:
            st["S"] = torch.zeros(H, d, dv, dtype=self.dtype)
            st["n"] = torch.zeros(H, d, dtype=self.dtype)
            st["m"] = [0.0] * H
        o = torch.empty(T, H, dv, dtype=self.dtype)
        for a in range(H):
            o[:, a], st["m"][a] = matrix_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a], st["S"][a], st["n"][a],
                                                st["m"][a])
        o = over_rms(o, self.eps).reshape(T, -1) * w[f"{p}.norm"] * torch.sigmoid(h @ w[f"{p}.g"].T)
        return o @ w[f"{p}.o"].T

    def linear(self, p, m, h, st):
        w, T = self.w, h.shape[0]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        q = (h @ w[f"{p}.q"].T).view(T, H, d) * d ** -0.5
        k, v = (h @ w[f"{p}.k"].T).view(T, H, d), (h @ w[f"{p}.v"].T).view(T, H, dv)
        z = (h @ w[f"{p}.a1"].T) @ w[f"{p}.a2"].T + w[f"{p}.a2.b"]
        alpha = torch.exp(F.logsigmoid(z) / m["tau"]).view(T, H, d)
        if "S" not in st:
            st["S"] = torch.zeros(H, d, dv, dtype=self.dtype)
        o = torch.stack([gated_linear(q[:, a], k[:, a], v[:, a], alpha[:, a], st["S"][a]) for a in range(H)], 1)
        o = (over_rms(o, self.eps) * w[f"{p}.norm"]).reshape(T, -1) * F.silu(h @ w[f"{p}.g"].T)
        return o @ w[f"{p}.o"].T

    def delta(self, p, m, h, st):
        w, T = self.w, h.shape[0]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        got = {}
        for x in ("q", "k", "v"):
            u = h @ w[f"{p}.{x}"].T
            before = st.get("conv." + x)
            if before is None:
                before = torch.zeros(m["conv"] - 1, u.shape[1], dtype=self.dtype)
            y, st["conv." + x] = causal_conv(u, w[f"{p}.{x}.conv"], before)
            got[x] = F.silu(y)
        q, k = unit(got["q"].view(T, G, d)) * d ** -0.5, unit(got["k"].view(T, G, d))
        v = got["v"].view(T, H, dv)
        beta = torch.sigmoid(h @ w[f"{p}.b"].T)
        g = torch.exp(-torch.exp(w[f"{p}.A_log"]) * F.softplus(h @ w[f"{p}.a"].T + w[f"{p}.dt_bias"]))
        if "S" not in st:
            st["S"] = torch.zeros(H, d, dv, dtype=self.dtype)
        rep = H // G
        o = torch.stack([delta_rule(q[:, a // rep], k[:, a // rep], v[:, a], beta[:, a], g[:, a], st["S"][a])
                         for a in range(H)], 1)
        o = over_rms(o, self.eps) * w[f"{p}.norm"]
        return (o.reshape(T, -1) * F.silu(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T

    def mixer(self, i, L, h, past, st):
        m, p = L["mixer"], f"l{i}.mix"
        if L["type"] == "delta":
            return self.delta(p, m, h, st)
        left, right = st.setdefault("left", {}), st.setdefault("right", {})
        if L["type"] == "parallel":
            a = self.biased_attention(f"{p}.left", m["left"], h, past, left)
            b = self.memory(f"{p}.right", m["right"], h, right)
        else:
            a = self.rotary_attention(f"{p}.left", m["left"], h, past, left)
            b = self.linear(f"{p}.right", m["right"], h, right)
        return m["left_scale"] * a + m["right_scale"] * b

    def feed_forward(self, p, h):
        w = self.w
        return (F.silu(h @ w[f"{p}.gate"].T) * (h @ w[f"{p}.up"].T)) @ w[f"{p}.down"].T

    # ---- one piece of one sequence ----
    def forward(self, toks: List[int], state: dict) -> torch.Tensor:
        w, r = self.w, self.cfg["residual_mult"]
        past = state["pos"]
        x = w["embed"][torch.tensor(toks)] * self.cfg["embedding"]["scale"]
        for i, L in enumerate(self.cfg["layers"]):
            h = layer_norm(x, w[f"l{i}.norm1"], self.eps)
            y = self.mixer(i, L, h, past, state["layers"][i]) * w[f"l{i}.ls1"]
            if L["mlp"]:
                y = y + self.feed_forward(f"l{i}.mlp", h) * w[f"l{i}.ls2"]
            x = x + r * y
            if self.taps is not None:
                self.taps.append(x.clone())
        state["pos"] = past + len(toks)
        return layer_norm(x, w["final.norm"], self.eps) @ w["embed"].T
