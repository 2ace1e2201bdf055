"""Saralix without a GPU: the configuration reader and its refusals, the spec it emits (tensor names and
shapes against the weights the tests make, cache needs), and the plain implementation against itself and
against closed forms -- each mechanism alone, a prompt whole against the same prompt in pieces down to
one token."""
import copy
import math

import pytest
import torch
import torch.nn.functional as F

from plain_saralix import (attend, causal_conv, clamped_glu, layer_norm, rotate_halves, route, ssm_scan, visible, yarn)
from saralix_helpers import CONFIGS, SARA_A, SARA_B, SARA_C, needle_model, needle_tokens, plain_logits, random_tokens, weights_of
from yalm_b200.cache import CacheNeed
from yalm_b200.config import ConfigError, architectures, config_from_dict
from yalm_b200.engine.lm import tensor_needs_of
from yalm_b200.parts import Model, Runtime
from yalm_b200.parts.position import yarn_frequencies


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


def test_parts_get_every_constant():
    assert "Saralix" in architectures()
    spec = config_from_dict(SARA_A).to_spec()
    p = spec.layers[0].part("mixer").params
    assert (p["num_heads"], p["head_dim"], p["rot_dim"], p["value_dim"], p["kv_rank"], p["scale"], p["rot_base"], p["window"],
            p["sink"], p["gate"], p["rot_layout"]) == (3, 24, 8, 16, 40, 0.2, 1e4, 33, True, None, "halves")
    assert p["rot_scaling"] == {"factor": 4.0, "original": 64, "fast": 32.0, "slow": 1.0} and p["eps"] == 1e-5
    f = spec.layers[0].part("feed_forward").params
    assert (f["intermediate_size"], f["limit"], f["slope"], f["shift"]) == (80, 1.5, 1.702, 1.0)
    m = spec.layers[1].part("mixer").params
    assert (m["num_heads"], m["head_dim"], m["state"], m["groups"], m["conv"], m["norm_groups"]) == (6, 20, 16, 3, 3, 2)
    e = spec.layers[1].part("feed_forward").params
    assert (e["experts"], e["top"], e["intermediate_size"], e["renormalise"]) == (6, 2, 40, True)
    c = spec.layers[2].part("mixer").params
    assert (c["window"], c["sink"], c["gate"]) == (None, False, "head")
    assert "feed_forward" not in spec.layers[2].parts
    assert config_from_dict(SARA_A).ignorable_tensor("l2.norm2b") and not config_from_dict(SARA_A).ignorable_tensor("l1.norm2")


def test_cache_needs():
    model = Model(config_from_dict(SARA_A).to_spec(), Runtime.shapes_only())
    needs = model.cache_needs()
    assert needs[(0, "mixer", "cache")] == CacheNeed("kv", kv_heads=1, head_dim=48, window=33, values=False)
    assert needs[(2, "mixer", "cache")] == CacheNeed("kv", kv_heads=1, head_dim=80, window=None, values=False)
    assert needs[(1, "mixer", "state")].state_shape == (6, 20, 16) and needs[(1, "mixer", "state")].state_dtype == torch.float32
    assert needs[(1, "mixer", "conv")].state_shape == (2, 120 + 2 * 3 * 16)
    assert model.step_flops([64], [0]) > 0 and model.step_bytes([50, 60]) > 0


@pytest.mark.parametrize("base, change, text", [
    (SARA_A, lambda d: d["layers"][0].update(type="window"), "type"),
    (SARA_A, lambda d: d["layers"][0]["mixer"].pop("mask"), "mask"),
    (SARA_A, lambda d: d["layers"][2]["mixer"].update(mask={"size": 4}), "mask"),
    (SARA_A, lambda d: d["layers"][0]["mixer"]["rot"].update(dims=4), "dims"),
    (SARA_A, lambda d: d["layers"][0]["mixer"].update(rot_dim=7), "rot_dim"),
    (SARA_A, lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (SARA_A, lambda d: d["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (SARA_A, lambda d: d["layers"][1]["mixer"].update(groups=4), "groups"),
    (SARA_A, lambda d: d["layers"][1]["mixer"].update(norm_groups=7), "norm_groups"),
    (SARA_A, lambda d: d["layers"][1]["mixer"].update(state=300), "state"),
    (SARA_A, lambda d: d["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (SARA_A, lambda d: d["layers"][1]["mlp"].update(kind="soft"), "kind"),
    (SARA_A, lambda d: d["layers"][0]["mlp"].pop("limit"), "limit"),
    (SARA_B, lambda d: d.pop("norm"), "norm"),
    (SARA_B, lambda d: d.update(layers=[]), "layers"),
])
def test_refusals(base, change, text):
    d = copy.deepcopy(base)
    change(d)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(d)


# ------------------------------------------------------------------ the plain implementation
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_against_pieces(name):
    cfg, seed = CONFIGS[name]
    w = weights_of(name)
    toks = random_tokens(41, cfg["vocab"], seed)
    ref, _ = plain_logits(cfg, w, toks)
    for pieces in ([1] * 41, [40, 1], [2, 5, 3]):
        got, _ = plain_logits(cfg, w, toks, pieces)
        assert torch.allclose(got, ref, atol=1e-5)
    other = list(toks)
    other[30] = (other[30] + 1) % cfg["vocab"]                             # causality
    got, _ = plain_logits(cfg, w, other)
    assert torch.allclose(got[:30], ref[:30], atol=1e-6) and not torch.allclose(got[30:], ref[30:], atol=1e-2)


def test_layer_norm_against_the_library_function():
    rnd = rnd_of(1)
    x, w = 3.0 + rnd(5, 30), rnd(30)
    assert torch.allclose(layer_norm(x, w, 1e-5), F.layer_norm(x, (30,), w, None, 1e-5))


def test_yarn_frequencies():
    scaling = {"factor": 8.0, "original": 512, "fast": 32.0, "slow": 1.0}
    f, mult = yarn(64, 1e4, scaling)
    plain, one = yarn(64, 1e4, None)
    assert one == 1.0 and mult == pytest.approx(0.1 * math.log(8.0) + 1.0)
    turns = 512 * plain / (2 * math.pi)
    assert torch.equal(f[turns > 40], plain[turns > 40])                   # fast pairs stay
    assert torch.allclose(f[turns < 0.8], plain[turns < 0.8] / 8.0)        # slow ones are slowed down
    between = (f < plain * 0.999) & (f > plain / 8.0 * 1.001)
    assert between.any()
    # ramps that collapse: fast and slow in one pair, all pairs above or below
    for dims, base, sc in ((2, 100.0, dict(scaling, original=4)), (8, 1e4, dict(scaling, fast=1.0)), (16, 1e6, dict(scaling, original=16)),
                           (64, 1e4, scaling), (24, 250.0, dict(scaling, factor=1.5, slow=0.5))):
        f, mult = yarn(dims, base, sc)
        g, m = yarn_frequencies(dims, base, sc)                            # the library's
        assert torch.allclose(f, g.double(), rtol=1e-6) and m == pytest.approx(mult)


def test_rotation_keeps_distances():
    rnd = rnd_of(2)
    f, _ = yarn(16, 1e4, None)
    q, k = rnd(1, 1, 16).expand(50, 1, 16), rnd(1, 1, 16).expand(50, 1, 16)
    pos = torch.arange(50)
    s = torch.einsum("ihd,jhd->ij", rotate_halves(q, pos, f, 1.3), rotate_halves(k, pos, f, 1.3))
    assert torch.allclose(s[10, 3], s[40, 33]) and torch.allclose(s[7, 7], 1.69 * (q[0, 0] * k[0, 0]).sum())


def test_masks_and_sinks():
    assert visible(3, 2, None).tolist() == [[True, True, True, False, False], [True] * 4 + [False], [True] * 5]
    assert visible(3, 2, 2).tolist() == [[False, True, True, False, False], [False, False, True, True, False],
                                         [False, False, False, True, True]]
    rnd = rnd_of(3)
    q, k, v = rnd(4, 2, 8), rnd(4, 2, 8), rnd(4, 2, 6)
    mask = visible(4, 0, 3)
    sink = torch.tensor([0.7, -2.0], dtype=torch.float64)
    # a sink is one more key of that score whose value is zero
    got = attend(q, k, v, mask, 0.4, sink)
    for h in range(2):
        s = (0.4 * q[:, h] @ k[:, h].T).masked_fill(~mask, float("-inf"))
        p = torch.softmax(torch.cat([s, sink[h].expand(4, 1)], 1), -1)[:, :4]
        assert torch.allclose(got[:, h], p @ v[:, h])
    assert torch.allclose(attend(q, k, v, mask, 0.4), attend(q, k, v, mask, 0.4, torch.full((2,), -1e4, dtype=torch.float64)))


def test_absorbed_form_of_the_latent_attention():
    """Queries moved into the latent space over the rows themselves, the mixed latent expanded after."""
    rnd = rnd_of(4)
    H, d, rd, dv, rank, T = 3, 8, 4, 6, 10, 9
    q, c, kr, uk, uv = rnd(T, H, d + rd), rnd(T, rank), rnd(T, rd), rnd(H, d, rank), rnd(H, dv, rank)
    k = torch.cat([torch.einsum("tr,hdr->thd", c, uk), kr[:, None].expand(T, H, rd)], -1)
    sink = rnd(H)
    ref = attend(q, k, torch.einsum("tr,hdr->thd", c, uv), visible(T, 0, 4), 0.3, sink)
    qa = torch.cat([torch.einsum("thd,hdr->thr", q[..., :d], uk), q[..., d:]], -1)
    rows = torch.cat([c, kr], -1)[:, None].expand(T, H, rank + rd)
    mixed = attend(qa, rows, c[:, None].expand(T, H, rank), visible(T, 0, 4), 0.3, sink)
    assert torch.allclose(torch.einsum("thr,hdr->thd", mixed, uv), ref)


def test_convolution_against_conv1d():
    rnd = rnd_of(5)
    u, w, b = rnd(20, 6), rnd(6, 4), rnd(6)
    ref = F.conv1d(F.pad(u.T[None], (3, 0)), w[:, None], b, groups=6)[0].T
    y, st = causal_conv(u, w, b, torch.zeros(3, 6, dtype=torch.float64))
    assert torch.allclose(y, ref) and torch.equal(st, u[-3:])
    y1, s1 = causal_conv(u[:2], w, b, torch.zeros(3, 6, dtype=torch.float64))
    y2, _ = causal_conv(u[2:], w, b, s1)
    assert torch.allclose(torch.cat([y1, y2]), ref)


def test_state_space_recurrence_as_one_sum():
    """y_t = sum_s exp(a_{s+1} + .. + a_t) dt_s (C_t . B_s) x_s + D x_t."""
    rnd = rnd_of(6)
    T, P, N = 12, 5, 7
    x, Bm, Cm, dt, a_log = rnd(T, P), rnd(T, N), rnd(T, N), rnd(T).abs(), torch.tensor(-0.5, dtype=torch.float64)
    S = torch.zeros(N, P, dtype=torch.float64)
    got = ssm_scan(x, Bm, Cm, dt, a_log, torch.tensor(0.3, dtype=torch.float64), S)
    la = torch.cumsum(-torch.exp(a_log) * dt, 0)
    m = torch.exp(la[:, None] - la[None, :]).tril() * (Cm @ Bm.T) * dt[None, :]
    assert torch.allclose(got, m @ x + 0.3 * x)


def test_feed_forwards():
    g, u = torch.tensor([5.0, -5.0, 1.0]).double(), torch.tensor([-9.0, 0.5, 9.0]).double()
    ref = [2 * torch.sigmoid(torch.tensor(3.404)) * (-1), -5 * torch.sigmoid(torch.tensor(-8.51)) * 1.5,
           1 * torch.sigmoid(torch.tensor(1.702)) * 3]
    assert torch.allclose(clamped_glu(g, u, 2.0), torch.tensor(ref).double(), atol=1e-6)     # gate clamped above only
    z = torch.tensor([0.1, 2.0, -1.0, 1.5]).double()
    chosen, w, margin = route(z, 2)
    assert chosen.tolist() == [1, 3] and margin == pytest.approx(1.4)
    full = torch.softmax(z, -1)[chosen]
    assert torch.allclose(w, full / full.sum())
    assert route(z, 4)[2] == float("inf")


@pytest.mark.parametrize("window", [None, 12])
def test_the_crafted_model_shows_a_lost_needle(window):
    cfg, w = needle_model(window)
    toks = needle_tokens(60, [20], [21, 31, 32, 59])
    blind = list(toks)
    blind[20] = 9
    ref, lost = plain_logits(cfg, w, toks)[0], plain_logits(cfg, w, blind)[0]
    for p in (21, 31, 32, 59):
        seen = window is None or p - 20 < window
        assert ((ref[p] - lost[p]).abs().max() > 0.4 * ref.abs().max()) == seen, p


def test_sizes_that_rule_out_the_aligned_paths():
    """The third configuration keeps off every 16-byte path: it is the one that tests the plain ones."""
    sizes = [v for L in SARA_C["layers"] for k, v in L["mixer"].items() if k in ("dim", "rot_dim", "vdim", "kv_rank", "state")]
    assert all(s % 8 for s in sizes) and SARA_C["width"] % 8
