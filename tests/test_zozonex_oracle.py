"""CPU: the plain Zozonex implementation against independent forms of each mechanism, and the reader of its config.json."""
import ctypes as C
import json

import numpy as np
import pytest

import lumi_b200
from lumi_b200 import synth, zozonex
from oracle import zozonex as oz


def rng(n):
    return np.random.default_rng(n)


def test_short_conv_is_a_causal_convolution():
    g = rng(0)
    x, w = g.standard_normal((19, 3)), g.standard_normal((3, 4))
    y = oz.short_conv(x, w)
    for c in range(3):
        assert np.allclose(y[:, c], np.convolve(x[:, c], w[c, ::-1])[:19])


def test_delta_rule_unrolled():
    """o_t as a sum over the writes that are left of every token, for a rule written without the state."""
    g = rng(1)
    T, dk, dv = 7, 5, 3
    q, k, v = g.standard_normal((T, dk)), oz.unit(g.standard_normal((T, dk))), g.standard_normal((T, dv))
    a, b = g.uniform(0.3, 1.0, T), g.uniform(0.1, 0.9, T)
    o, S = oz.delta_rule(q, k, v, a, b)
    # S_t = g_t (I - b_t k_t k_t^T) S_{t-1} + b_t k_t v_t^T
    M = np.zeros((dk, dv))
    for t in range(T):
        M = a[t] * (np.eye(dk) - b[t] * np.outer(k[t], k[t])) @ M + b[t] * np.outer(k[t], v[t])
        assert np.allclose(o[t], M.T @ q[t])
    assert np.allclose(S, M)


def test_sink_is_one_more_score_without_a_value():
    s = rng(2).standard_normal((4, 6)) * 30
    full = np.concatenate([np.zeros((4, 1)), s], axis=1)
    e = np.exp(full - full.max(1, keepdims=True))
    assert np.allclose(oz.softmax_with_sink(s), (e / e.sum(1, keepdims=True))[:, 1:])
    assert np.all(oz.softmax_with_sink(np.full((1, 3), -200.0)) < 1e-80)


def test_window_counts_the_token_itself():
    m = oz.window_mask(6, 3)
    assert [list(np.flatnonzero(r)) for r in m] == [[0], [0, 1], [0, 1, 2], [1, 2, 3], [2, 3, 4], [3, 4, 5]]


def test_position_vector():
    p = oz.sinusoid([0, 5], 6)
    assert np.allclose(p[0], [0, 1, 0, 1, 0, 1])
    assert np.allclose(p[1, 2:4], [np.sin(5 * 10000 ** (-2 / 6)), np.cos(5 * 10000 ** (-2 / 6))])


def test_layers_can_read_an_earlier_layers_keys():
    """With equal query and output weights a sharing layer repeats its source's attention for the same input."""
    g = rng(3)
    h = g.standard_normal((9, 12))
    W = {"q": g.standard_normal((8, 12)), "k": g.standard_normal((4, 12)), "v": g.standard_normal((6, 12)), "o": g.standard_normal((12, 12))}
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 6, "mask": {"size": 4}, "scale": 0.7}
    y, kv = oz.attention_mixer(W, "", m, h, 1e-5, {})
    W2 = {n: W[n] for n in ("q", "o")}
    z, _ = oz.attention_mixer(W2, "", dict(m, kv_from=0), h, 1e-5, {0: kv})
    assert np.allclose(y, z)


def small():
    return zozonex.config(40, 50, [zozonex.delta(2, 8, 12, kv_heads=1, ff=24), zozonex.attention(4, 8, 5, vdim=12, kv_heads=2),
                                   zozonex.attention(4, 8, 9, vdim=12, kv_heads=2, ff=16, kv_from=1)], eps=1e-4, embed_scale=3.0)


def test_forward_is_causal():
    cfg = small()
    W = {n: synth.as_f32(dt, a) for n, dt, a in zozonex.iter_tensors(cfg, seed=1)}
    toks = list(rng(4).integers(0, 50, 20))
    a = oz.forward(cfg.raw, W, toks)[0]
    toks[12] = (toks[12] + 1) % 50
    b = oz.forward(cfg.raw, W, toks)[0]
    assert np.allclose(a[:12], b[:12]) and not np.allclose(a[12], b[12])


def _create(text):
    h = C.c_void_p()
    st = lumi_b200.lib().lumi_model_create(text.encode(), 0, C.byref(h))
    msg = lumi_b200.lib().lumi_last_error().decode()
    if st == 0:
        lumi_b200.lib().lumi_model_free(h)
    return st, msg


def test_good_config_is_read():
    st, msg = _create(small().to_json())
    assert st in (0, -6), msg                # OK on a GPU box, LUMI_E_CUDA where no device exists
    assert isinstance(synth.config_from_json(small().to_json()), zozonex.ZozonexConfig)
    assert isinstance(synth.config_from_json(synth.tiny_config().to_json()), synth.ModelConfig)


@pytest.mark.parametrize("change,frag", [
    (lambda c: c.update(architecture="Nothing"), "not known"),
    (lambda c: c.pop("width"), "'width'"),
    (lambda c: c["norm"].pop("eps"), "'eps'"),
    (lambda c: c.update(layers=[]), "non-empty"),
    (lambda c: c["layers"][0].update(type="other"), "not known"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "not divisible"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "'conv'"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "'scale'"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), ">= 1"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "earlier layer"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "no keys and values"),
    (lambda c: c["layers"][2]["mixer"].update(dim=6), "head sizes differ"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "feed-forward kind"),
])
def test_bad_config_is_rejected(change, frag):
    raw = json.loads(small().to_json())
    change(raw)
    st, msg = _create(json.dumps(raw))
    assert st == -2 and frag in msg, (st, msg)
