"""Tetodra without a GPU: the configuration reader and its refusals, the spec it emits (tensor names and
shapes against the weights the tests make, cache needs), and the plain implementation against itself and
against closed forms -- each mechanism alone, a prompt whole against the same prompt in pieces down to
one token."""
import copy
import math

import pytest
import torch
import torch.nn.functional as F

from plain_tetodra import (attend, causal_conv, delta_rule, distance_bucket, gated_linear, layer_norm, matrix_memory,
                           query_temperature, rotate_halves, unit)
from tetodra_helpers import (CONFIGS, NEEDLE, TET_A, TET_B, TET_C, needle_model, needle_tokens, plain_logits,
                             random_tokens, weights_of)
from yalm_b200.cache import Cache, CacheNeed
from yalm_b200.config import ConfigError, architectures, config_from_dict
from yalm_b200.engine.lm import tensor_needs_of
from yalm_b200.parts import Model, Runtime
from yalm_b200.parts.exact_attention import distance_buckets
from yalm_b200.parts.linear import stacked_rows


def rnd_of(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *shape: torch.randn(*shape, generator=g, dtype=torch.float64)


# ------------------------------------------------------------------ configuration
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_spec_names_the_tests_weights(name):
    cfg, w = config_from_dict(CONFIGS[name][0]), weights_of(name)
    needs = tensor_needs_of(cfg)
    assert sorted(needs) == sorted(w)
    for k, need in needs.items():
        assert tuple(need.shape) == tuple(w[k].shape), k
    spec = cfg.to_spec()
    assert [e.layer for e in spec.run_order] == list(range(len(cfg.layers)))
    assert spec.head.tensors["weight"] == spec.embedding.tensors["weight"] == "embed"
    assert config_from_dict(cfg.to_dict()) == cfg


def test_sizes_that_only_tensors_give():
    """Without the two sizes in the configuration they come from the checkpoint's shapes."""
    d = copy.deepcopy(TET_A)
    for ld in d["layers"]:
        for side in ("left", "right"):
            for k in ("bias_rows", "decay_rank"):
                (ld["mixer"].get(side) or {}).pop(k, None)
    w = weights_of("tet_a")
    cfg = config_from_dict(d).with_tensor_shapes({k: tuple(v.shape) for k, v in w.items()})
    assert [l.bias_rows for l in cfg.layers if l.kind == "parallel"] == [10]
    assert [l.decay_rank for l in cfg.layers if l.kind == "parallel_2"] == [12, 5]
    for k, need in tensor_needs_of(cfg).items():
        assert tuple(need.shape) == tuple(w[k].shape), k


def test_parts_get_every_constant():
    assert "Tetodra" in architectures()
    spec = config_from_dict(TET_A).to_spec()
    assert spec.embedding.params["scale"] == 3.0
    p = spec.layers[0].part("mixer").params
    assert p["scales"] == [0.8, 0.7] and [n for n, _ in p["branches"]] == ["left", "right"]
    left, right = (s.params for _, s in p["branches"])
    assert (left["num_heads"], left["num_kv_heads"], left["head_dim"], left["value_dim"], left["scale"]) == (6, 2, 24, 40, 0.25)
    assert left["rotation"] == {"dims": 16, "base": 1e4}
    assert (right["num_heads"], right["key_dim"], right["value_dim"], right["tau"], right["decay_rank"]) == (3, 20, 36, 8.0, 12)
    d = spec.layers[1].part("mixer").params
    assert (d["num_heads"], d["num_kv_heads"], d["key_dim"], d["value_dim"], d["conv"], d["decay"], d["gate"]) == (
        4, 2, 32, 24, 4, "head", "silu")
    left, right = (s.params for _, s in spec.layers[2].part("mixer").params["branches"])
    assert left["distance_bias"] == {"rows": 10, "largest": 50.0} and left["q_temperature"] == {"coef": 0.25, "every": 16.0}
    assert left["sink"] and left["values_from_keys"] and left["qk_head_norm"] == {"eps": 1e-5}
    assert (right["num_heads"], right["key_dim"], right["value_dim"], right["gate_cap"]) == (3, 16, 28, 7.0)
    assert spec.layers[0].part("mixer_scale").params["factor"] == spec.layers[0].part("feed_forward_scale").params["factor"] == 0.8
    assert "feed_forward" not in spec.layers[3].parts
    cfg = config_from_dict(TET_A)
    assert cfg.ignorable_tensor("l3.ls2") and not cfg.ignorable_tensor("l2.ls2")


def test_cache_needs():
    model = Model(config_from_dict(TET_A).to_spec(), Runtime.shapes_only())
    needs = model.cache_needs()
    assert needs[(0, "mixer", "left.cache")] == CacheNeed("kv", kv_heads=2, head_dim=24, value_dim=40)
    assert needs[(0, "mixer", "right.cache")].state_shape == (3, 36, 20)
    assert needs[(1, "mixer", "state")].state_shape == (4, 24, 32)
    assert needs[(1, "mixer", "conv")].state_shape == (3, 2 * 2 * 32 + 4 * 24)
    assert needs[(2, "mixer", "right.state")].state_shape == (3, 32, 16)          # 28 values, n and padding
    assert needs[(2, "mixer", "right.maximum")].state_shape == (3,)
    assert all(n.state_dtype == torch.float32 for n in needs.values() if n.kind == "state")
    assert model.step_flops([64], [0]) > 0 and model.step_bytes([50, 60]) > 0


@pytest.mark.parametrize("max_tokens", [None, 256])
def test_cache_keeps_values_of_their_own_size(max_tokens):
    needs = {("a",): CacheNeed("kv", kv_heads=2, head_dim=8, value_dim=24), ("b",): CacheNeed("kv", kv_heads=2, head_dim=8)}
    c = Cache(needs, 4, 512, torch.float32, "cpu", max_tokens=max_tokens)
    assert len(c.groups) == 2
    v = c.view(("a",))
    assert v.k.shape[-1] == 8 and v.v.shape[-1] == 24 and v.k.shape[:-1] == v.v.shape[:-1]
    assert c.view(("b",)).v.shape[-1] == 8
    assert c.bytes() == Cache.bytes_needed(needs, 4, 512, torch.float32, max_tokens)


@pytest.mark.parametrize("base, change, text", [
    (TET_A, lambda d: d["layers"][0].update(type="window"), "type"),
    (TET_A, lambda d: d["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (TET_A, lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=4), "kv_heads"),
    (TET_A, lambda d: d["layers"][0]["mixer"]["left"].update(vdim=300), "vdim"),
    (TET_A, lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=26), "dims"),
    (TET_A, lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "dims"),
    (TET_A, lambda d: d["layers"][0]["mixer"]["right"].pop("tau"), "tau"),
    (TET_A, lambda d: d["layers"][0]["mixer"]["right"].update(dim=300), "dim"),
    (TET_A, lambda d: d["layers"][1]["mixer"].update(conv=1), "taps"),
    (TET_A, lambda d: d["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (TET_A, lambda d: d["layers"][2]["mixer"]["left"].update(vdim=16), "vdim"),
    (TET_A, lambda d: d["layers"][2]["mixer"]["left"].pop("bias_max"), "bias_max"),
    (TET_A, lambda d: d["layers"][2]["mixer"]["left"]["q_temp"].update(every=0), "every"),
    (TET_A, lambda d: d["layers"][2]["mixer"]["right"].pop("gate_cap"), "gate_cap"),
    (TET_A, lambda d: d["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (TET_B, lambda d: d.pop("norm"), "norm"),
    (TET_B, lambda d: d.update(layers=[]), "layers"),
])
def test_refusals(base, change, text):
    d = copy.deepcopy(base)
    change(d)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(d)


def test_a_table_that_cannot_be_is_refused_by_its_part():
    with pytest.raises(ValueError, match="distance table"):
        distance_buckets(16, 8)


# ------------------------------------------------------------------ the plain implementation
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_against_pieces(name):
    cfg, seed = CONFIGS[name]
    w = weights_of(name)
    toks = random_tokens(41, cfg["vocab"], seed)
    ref = plain_logits(cfg, w, toks)
    for pieces in ([1] * 41, [40, 1], [2, 5, 3]):
        assert torch.allclose(plain_logits(cfg, w, toks, pieces), ref, atol=1e-5)
    other = list(toks)
    other[30] = (other[30] + 1) % cfg["vocab"]                             # causality
    got = plain_logits(cfg, w, other)
    assert torch.allclose(got[:30], ref[:30], atol=1e-6) and not torch.allclose(got[30:], ref[30:], atol=1e-2)


def test_layer_norm_and_convolution_against_the_library_functions():
    rnd = rnd_of(1)
    x, w = 3.0 + rnd(5, 30), rnd(30)
    assert torch.allclose(layer_norm(x, w, 1e-5), F.layer_norm(x, (30,), w, None, 1e-5))
    u, c = rnd(9, 4), rnd(4, 3)
    y, before = causal_conv(u, c, torch.zeros(2, 4, dtype=torch.float64))
    assert torch.allclose(y, F.conv1d(F.pad(u.T[None], (2, 0)), c[:, None], groups=4)[0].T) and torch.equal(before, u[-2:])
    assert torch.allclose(unit(x).norm(dim=-1), torch.ones(5, dtype=torch.float64), atol=1e-6)


@pytest.mark.parametrize("rows, largest", [(16, 120), (32, 128), (2, 7), (10, 50), (16, 128), (7, 1000), (33, 17)])
def test_distance_buckets(rows, largest):
    """The near half has a row per distance, rows grow with the distance, the last begins where the rule says
    and holds for good; a table of powers of two has its edges exactly there."""
    table = distance_buckets(rows, largest)
    far = 3 * int(largest)
    for n in range(far):
        assert (table[n] if n < len(table) else table[-1]) == distance_bucket(n, rows, largest), n
    assert table[:rows // 2] == list(range(rows // 2)) and table == sorted(table) and table[-1] == rows - 1
    if (rows, largest) == (16, 128):                  # 8 * 2^(k / 2): 8, 11.3, 16, 22.6, 32, 45.3, 64, 90.5
        assert [table.index(8 + k) for k in range(8)] == [8, 12, 16, 23, 32, 46, 64, 91]
    if (rows, largest) == (2, 7):                     # one row for distance 0, one for all others
        assert table == [0, 1]


def test_temperature():
    assert query_temperature(0, 0.5, 4) == 1.0 and query_temperature(2, 0.5, 4) == 1.0
    assert query_temperature(3, 0.5, 4) == pytest.approx(1.0 + 0.5 * math.log(2))
    assert query_temperature(0, 0.5, 1) == pytest.approx(1.0 + 0.5 * math.log(2))


def test_attention_with_bias_and_sink():
    rnd = rnd_of(3)
    q, k, v = rnd(6, 4, 8), rnd(6, 2, 8), rnd(6, 2, 5)
    ref = F.scaled_dot_product_attention(q.transpose(0, 1), k.repeat_interleave(2, 1).transpose(0, 1),
                                         v.repeat_interleave(2, 1).transpose(0, 1), is_causal=True, scale=0.3)
    assert torch.allclose(attend(q, k, v, 0, 0.3), ref.transpose(0, 1))
    # a bias shared by all keys changes nothing without a sink, a sink of the same size does
    flat = torch.full((4, 6, 6), 2.0, dtype=torch.float64)
    assert torch.allclose(attend(q, k, v, 0, 0.3, bias=flat), ref.transpose(0, 1))
    sink = torch.full((4,), 100.0, dtype=torch.float64)
    assert attend(q, k, v, 0, 0.3, sink=sink).abs().max() < 1e-20
    # the sink counts once: one key with score 0 and a sink of ln 3 leave it a quarter
    one = attend(torch.zeros(1, 1, 2).double(), torch.zeros(1, 1, 2).double(), torch.ones(1, 1, 1).double(), 0, 1.0,
                 sink=torch.tensor([math.log(3.0)], dtype=torch.float64))
    assert float(one) == pytest.approx(0.25)


def test_rotation_depends_on_distance_alone():
    rnd = rnd_of(4)
    q, k = rnd(1, 1, 12), rnd(1, 1, 12)
    dots = [float((rotate_halves(q, torch.tensor([p + 7]), 8, 100.0) * rotate_halves(k, torch.tensor([p]), 8, 100.0)).sum())
            for p in (0, 3, 500)]
    assert dots[0] == pytest.approx(dots[1]) and dots[0] == pytest.approx(dots[2])
    assert torch.equal(rotate_halves(q, torch.tensor([9]), 8, 100.0)[..., 8:], q[..., 8:])


def test_matrix_memory_without_a_running_maximum():
    """The maximum is only a common factor: the outputs are those of the sums without it, but for the floor, which
    is exp(-m), and the 1e-6."""
    rnd = rnd_of(5)
    T, dk, dv = 12, 4, 3
    q, k, v = rnd(T, dk), rnd(T, dk), rnd(T, dv)
    i, f = 3.0 * rnd(T), F.logsigmoid(2.0 * rnd(T))
    S, n = torch.zeros(dk, dv).double(), torch.zeros(dk).double()
    o, m = matrix_memory(q, k, v, i, f, S, n, 0.0)
    S2, n2, m2 = torch.zeros(dk, dv).double(), torch.zeros(dk).double(), 0.0
    for t in range(T):
        S2 = math.exp(f[t]) * S2 + math.exp(i[t]) * torch.outer(k[t], v[t])
        n2 = math.exp(f[t]) * n2 + math.exp(i[t]) * k[t]
        m2 = max(float(f[t]) + m2, float(i[t]))
        ref = S2.T @ q[t] / (max(abs(float(n2 @ q[t])), 1.0) + 1e-6 * math.exp(m2))
        assert torch.allclose(o[t], ref, rtol=1e-9), t
    assert m == pytest.approx(m2) and torch.allclose(S * math.exp(m), S2)


def test_linear_recurrences_against_sums():
    rnd = rnd_of(6)
    T, dk, dv = 9, 3, 2
    q, k, v = rnd(T, dk), rnd(T, dk), rnd(T, dv)
    alpha = torch.sigmoid(rnd(T, dk))
    o = gated_linear(q, k, v, alpha, torch.zeros(dk, dv).double())
    for t in range(T):
        ref = sum(((q[t] * alpha[s + 1:t + 1].prod(0) * k[s]).sum()) * v[s] for s in range(t + 1))
        assert torch.allclose(o[t], ref)
    # orthonormal keys, beta 1, no decay: a key's value is read back whatever else was written
    keys = torch.eye(4, dtype=torch.float64)
    vals = rnd(4, dv)
    S = torch.zeros(4, dv).double()
    one = torch.ones(4).double()
    delta_rule(keys, keys, vals, one, one, S)
    assert torch.allclose(S, vals)
    delta_rule(keys[:1], keys[:1], rnd(1, dv), one[:1], one[:1], S)          # a second write replaces the first
    assert not torch.allclose(S[0], vals[0]) and torch.allclose(S[1:], vals[1:])
    delta_rule(keys[1:2], keys[1:2], vals[1:2], one[:1], 0.5 * one[:1], S)
    assert torch.allclose(S[1], vals[1]) and torch.allclose(S[2:], 0.5 * vals[2:])


@pytest.mark.parametrize("kind", ["parallel", "parallel_2"])
def test_a_needle_decides(kind):
    cfg, w = needle_model(kind)
    at, n = 20, 150
    near, mid, far = at + 5, at + 15, at + 100
    toks = needle_tokens(n, [at], [near, mid, far])
    blind = list(toks)
    blind[at] = 9
    ref, lost = plain_logits(cfg, w, toks), plain_logits(cfg, w, blind)
    for p, seen in ((near, True), (mid, kind == "parallel_2"), (far, True)):
        assert ((ref[p] - lost[p]).abs().max() > 0.4 * ref[near].abs().max()) == seen, (kind, p)
        if seen:
            assert ref[p].argmax() == NEEDLE


def test_stacked_rows():
    a, b, c = torch.ones(3, 5), 2 * torch.ones(4, 5), 3 * torch.ones(2, 5)
    w, first = stacked_rows([a, b, c])
    assert first == [0, 4, 8] and w.shape == (12, 5)
    assert w[3].abs().max() == 0 and torch.equal(w[4:8], b) and torch.equal(w[8:10], c)
