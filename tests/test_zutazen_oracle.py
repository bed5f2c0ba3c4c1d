"""CPU: the plain Zutazen implementation against independent forms of each mechanism, and the reader of its config.json."""
import ctypes as C
import json

import numpy as np
import pytest

import lumi_b200
from lumi_b200 import synth, zutazen as zt
from oracle import zutazen as oz


def rng(n):
    return np.random.default_rng(n)


def test_retention_unrolled():
    """o_t as a sum over all earlier tokens, without the state."""
    g = rng(0)
    q, k, v, d = g.standard_normal((9, 4)), g.standard_normal((9, 4)), g.standard_normal((9, 3)), 0.83
    o, S = oz.retention(q, k, v, d)
    for t in range(9):
        assert np.allclose(o[t], sum(d ** (t - s) * (q[t] @ k[s]) * v[s] for s in range(t + 1)))
    assert np.allclose(S, sum(d ** (8 - s) * np.outer(k[s], v[s]) for s in range(9)))
    assert np.allclose(oz.retention(q, k, v, 0.0)[0], (q * k).sum(1)[:, None] * v)


@pytest.mark.parametrize("rotate", [oz.rotate_half, oz.rotate_pairs])
def test_rotation_keeps_relative_positions(rotate):
    """Scores of rotated vectors depend on the distance alone; dimensions beyond `dims` stay; position 0 does not turn."""
    g = rng(1)
    q, k = g.standard_normal(10), g.standard_normal(10)
    at = lambda x, p: rotate(x[None], 6, 50.0, first=p)[0]
    assert np.allclose(at(q, 0), q) and np.allclose(at(q, 77)[6:], q[6:])
    assert np.isclose(at(q, 30) @ at(k, 21), at(q, 9) @ at(k, 0))
    assert not np.isclose(at(q, 30) @ at(k, 21), at(q, 30) @ at(k, 20))


def test_rotation_layouts():
    x = np.arange(1.0, 7.0)
    c, s = oz.rotation([2], 4, 9.0)
    half, pairs = oz.rotate_half(x[None], 4, 9.0, first=2)[0], oz.rotate_pairs(x[None], 4, 9.0, first=2)[0]
    assert np.isclose(c[0, 1], np.cos(2 * 9.0 ** -0.5))
    assert np.allclose(half[[0, 2]], [1 * c[0, 0] - 3 * s[0, 0], 3 * c[0, 0] + 1 * s[0, 0]])
    assert np.allclose(pairs[[2, 3]], [3 * c[0, 1] - 4 * s[0, 1], 4 * c[0, 1] + 3 * s[0, 1]])


def test_conv_is_causal():
    g = rng(2)
    x, w, b = g.standard_normal((11, 3)), g.standard_normal((3, 4)), g.standard_normal(3)
    y = oz.causal_conv(x, w, b)
    for c in range(3):
        assert np.allclose(y[:, c], b[c] + np.convolve(x[:, c], w[c, ::-1])[:11])


def test_block_linear_is_a_block_diagonal_matrix():
    g = rng(3)
    w, b, u = g.standard_normal((3, 4, 4)), g.standard_normal((3, 4)), g.standard_normal((5, 12))
    full = np.zeros((12, 12))
    for i in range(3):
        full[4 * i:4 * i + 4, 4 * i:4 * i + 4] = w[i]
    assert np.allclose(oz.block_linear(w, b, u), u @ full.T + b.reshape(-1))


def test_linear_recurrence_unrolled():
    g = rng(4)
    u, r, i, lam = g.standard_normal((7, 2)), g.uniform(0, 1, (7, 2)), g.uniform(0, 1, (7, 2)), g.uniform(-3, 1, 2)
    a = np.exp(-8 * r * np.log1p(np.exp(lam)))
    S = oz.rglru(u, r, i, lam)
    for t in range(7):
        assert np.allclose(S[t], sum(np.prod(a[s + 1:t + 1], axis=0) * np.sqrt(1 - a[s] ** 2) * i[s] * u[s] for s in range(t + 1)))


def test_window_counts_the_token_itself():
    v = np.eye(6)[:, None, :]
    o = oz.window_attention(np.zeros((6, 1, 2)), np.zeros((6, 1, 2)), v, 1.0, 3)[:, 0]
    assert np.allclose(o[5], [0, 0, 0, 1 / 3, 1 / 3, 1 / 3]) and np.allclose(o[1], [0.5, 0.5, 0, 0, 0, 0])


def test_latent_queries_can_be_absorbed():
    """q.(U c) = (U^T q).c and sum p (V c) = V (sum p c): what lets all heads share the cached rows."""
    g = rng(5)
    U, V, q, c = g.standard_normal((4, 6)), g.standard_normal((3, 6)), g.standard_normal(4), g.standard_normal((9, 6))
    p = g.uniform(0, 1, 9)
    assert np.allclose((c @ U.T) @ q, c @ (U.T @ q)) and np.allclose(p @ (c @ V.T), V @ (p @ c))


def test_routing():
    chosen, w = oz.route(np.array([[0.0, 3.0, -1.0, 2.0], [1.0, 1.0, 0.0, 1.0]]), 2)
    assert [list(c) for c in chosen] == [[1, 3], [0, 1]]                    # equal scores: the lower index
    assert np.allclose(w, 1 / (1 + np.exp(-np.array([[3.0, 2.0], [1.0, 1.0]]))))      # not renormalised


def test_the_weight_multiplies_the_experts_input():
    g = rng(6)
    W = {"x.router": g.standard_normal((2, 5))}
    for e in range(2):
        for n, s in (("gate", (3, 5)), ("up", (3, 5)), ("down", (5, 3))):
            W["x.e%d.%s" % (e, n)] = g.standard_normal(s)
    h = g.standard_normal((1, 5))
    y = oz.moe_mlp(W, "x.", {"router": {"top": 2}}, h)
    s = 1 / (1 + np.exp(-(W["x.router"] @ h[0])))
    ref = np.zeros(5)
    for e in range(2):
        a = W["x.e%d.gate" % e] @ (s[e] * h[0])
        ref += W["x.e%d.down" % e] @ (a / (1 + np.exp(-a)) * (W["x.e%d.up" % e] @ (s[e] * h[0])))
    assert np.allclose(y[0], ref)


def small():
    layers = [zt.retention(2, 8, 6, mlp=zt.moe(3, 2, 10)), zt.rglru(24, 2, conv=3), zt.latent_attention(2, 6, 4, 5, 12, 7, mlp=zt.dense(20))]
    layers.append(zt.again(layers, 0))
    return zt.config(40, 50, layers, embed_scale=3.0)


def test_layers_with_another_layers_weights():
    """A layer that names another one computes what a copy of its tensors would."""
    cfg = small()
    W = {n: synth.as_f32(dt, a) for n, dt, a in zt.iter_tensors(cfg, seed=1)}
    copy = zt.config(40, 50, cfg.raw["layers"][:3] + [cfg.raw["layers"][0]], embed_scale=3.0)
    W2 = dict(W, **{"l3." + n[3:]: a for n, a in W.items() if n.startswith("l0.")})
    toks = [1, 4, 9, 2, 30]
    assert np.array_equal(oz.forward(cfg.raw, W, toks)[0], oz.forward(copy.raw, W2, toks)[0])
    assert not any(n.startswith("l3.") for n in W)


def parse(raw):
    h = C.c_void_p()
    rc = lumi_b200.lib().lumi_model_create(json.dumps(raw).encode(), 0, C.byref(h))
    msg = lumi_b200.lib().lumi_last_error().decode()
    if rc == 0:
        lumi_b200.lib().lumi_model_free(h)
    return rc, msg


@pytest.mark.parametrize("where,key,value,text", [
    (("layers", 0, "mixer"), "decay", [0.5], "one number per head"), (("layers", 0, "mixer"), "decay", [0.5, 1.5], "[0, 1]"),
    (("layers", 0, "mixer", "rot"), "dims", 3, "even"), (("layers", 0, "mixer", "rot"), "dims", 10, "exceeds dim"),
    (("layers", 1, "mixer"), "blocks", 5, "not divisible"), (("layers", 2, "mixer", "rot"), "dims", 6, "rot_dim"),
    (("layers", 2, "mixer"), "kv_rank", None, "kv_rank"), (("layers", 0, "mlp", "router"), "top", 4, "exceeds"),
    (("layers", 3), "weights_of", 3, "earlier"), (("layers", 3), "weights_of", 1, "sizes differ"), (("layers", 1), "type", "other", "not known"),
    (("layers", 2, "mlp"), "kind", "other", "not known"), (("norm",), "eps", None, "eps")])
def test_reader_refuses(where, key, value, text):
    raw = json.loads(small().to_json())
    at = raw
    for w in where:
        at = at[w]
    if value is None:
        del at[key]
    else:
        at[key] = value
    rc, msg = parse(raw)
    assert rc == -2 and text in msg, (rc, msg)


def test_reader_takes_the_design():
    rc, msg = parse(json.loads(small().to_json()))
    assert rc == 0 or rc == -6, msg                                          # -6: no CUDA device on this machine
    assert synth.config_from_json(small().to_json()).d_model == 40
