"""GPU: the Zutazen design — each mechanism alone (models of one layer), then whole models through the session API — against the
plain implementation in oracle/zutazen.py."""
import json
import os
import subprocess

import numpy as np
import pytest

import lumi_b200
from lumi_b200 import synth, zutazen as zt
from oracle import zutazen as oz

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {True: 1e-4, False: 3e-2}      # fp32 / bf16 weights and cache; worst logit over the logits' root mean square


def rel(got, ref):
    """Error of rows relative to the reference's root mean square."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    return float(np.abs(got - ref).max() / np.sqrt((ref ** 2).mean()))


def cuts(T, sizes):
    out, at = [], 0
    while at < T:
        n = min(sizes[len(out) % len(sizes)], T - at)
        out.append((at, n))
        at += n
    return out


def weights(tens):
    return {n: synth.as_f32(dt, a) for n, dt, a in tens}


def replace(tens, **changes):
    """Tensors by name (dots as double underscores) replaced by other values, as bf16."""
    by = {k.replace("__", "."): v for k, v in changes.items()}
    assert set(by) <= {n for n, _, _ in tens}
    return [(n, dt, synth.f32_to_bf16_bits(np.asarray(by[n], np.float32).reshape(a.shape)) if n in by else a) for n, dt, a in tens]


def run(sess, toks, sizes, slot=0):
    sess.reset([slot])
    return np.concatenate([sess.extend(toks[at:at + n], range(n), slot=slot) for at, n in cuts(len(toks), sizes)])


# ---- each mechanism alone --------------------------------------------------------------------------------------------
ALONE = {
    # heads whose state fits a few registers, many, the state in global memory (and beyond the chunked form); rotated in part, not at
    # all; decays of one, nearly one, one half and zero; sizes off every vector width
    "retention": [zt.retention(3, 24, 36, [1.0, 0.5, 0.999], rot_dims=16, base=300.0)],
    "retention_wide": [zt.retention(2, 128, 128)],
    "retention_odd": [zt.retention(1, 33, 130, [0.97], rot_dims=0), zt.retention(2, 20, 7, [0.0, 0.9], rot_dims=2)],
    "retention_tall": [zt.retention(1, 250, 40, [0.98], rot_dims=100)],
    "retention_huge": [zt.retention(1, 300, 280, [0.99])],
    # blocks off every tile, one block, blocks of one channel; filters of several lengths and of a single tap
    "rglru": [zt.rglru(88, 4, conv=3)],
    "rglru_one_block": [zt.rglru(160, 1, conv=2)],
    "rglru_long_filter": [zt.rglru(45, 3, conv=7)],
    "rglru_single_tap": [zt.rglru(64, 64, conv=1)],
    # more heads than a tile holds; a latent of full size; no rotated part; windows of one token, around a page, none
    "latent": [zt.latent_attention(3, 20, 12, 28, 40, 37, base=200.0)],
    "latent_many_heads": [zt.latent_attention(19, 8, 4, 6, 72, 64)],
    "latent_large": [zt.latent_attention(5, 96, 64, 128, 512, 130)],
    "latent_larger": [zt.latent_attention(2, 40, 30, 24, 700, 65)],
    "latent_wide_heads": [zt.latent_attention(2, 250, 16, 264, 48, 50)],
    "latent_unrotated": [zt.latent_attention(2, 48, 0, 40, 64, 1)],
    "latent_all": [zt.latent_attention(4, 32, 16, 32, 96, 0, scale=0.3)],
}


def alone(name, seed=3):
    width = {"retention_odd": 40, "latent_many_heads": 72, "latent_large": 192}.get(name, 64)
    cfg = zt.config(width, 90, ALONE[name], eps=3e-5, embed_scale=2.0)
    return cfg, list(zt.iter_tensors(cfg, seed=seed))


@pytest.mark.parametrize("fp32", [True, False])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mixer_alone(name, fp32):
    """The whole prompt, single tokens, and uneven portions (down to two tokens, on both sides of what goes by chunks)."""
    cfg, tens = alone(name)
    toks = np.random.default_rng(len(name)).integers(0, 90, 210).astype(np.uint32)
    ref = oz.forward(cfg.raw, weights(tens), toks)[0]
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    sess = model.init_states(2, 256)
    for slot, sizes in ((0, [210]), (1, [1]), (1, [70, 2, 3, 1, 17, 15, 16]), (0, [9])):
        got = run(sess, toks, sizes, slot)
        assert rel(got, ref) < TOL[fp32], (slot, sizes, rel(got, ref))
    sess.close(); model.close()


FF = {"dense": zt.dense(56), "dense_wide": zt.dense(330), "top1": zt.moe(7, 1, 24), "top3": zt.moe(40, 3, 20), "all": zt.moe(5, 5, 72),
      "single": zt.moe(1, 1, 33), "many": zt.moe(300, 2, 16)}


@pytest.mark.parametrize("fp32", [True, False])
@pytest.mark.parametrize("name", sorted(FF))
def test_feed_forward_alone(name, fp32):
    """A mixer that adds nothing: the feed-forward sees the embedding, so the choice of experts is known per token; few rows, many
    rows, and batches in which some experts get no token."""
    cfg = zt.config(72, 120, [zt.rglru(8, 1, mlp=FF[name])], embed_scale=2.0)
    tens = list(zt.iter_tensors(cfg, seed=5))
    tens = replace(tens, l0__mix__o=np.zeros((72, 8)))
    W = weights(tens)
    if FF[name]["kind"] == "moe":
        ids = [t for t in range(120) if router_margin(cfg, W, t) > 1e-3]
        assert len(ids) > 60
    else:
        ids = list(range(120))
    toks = np.random.default_rng(1).choice(ids, 300).astype(np.uint32)
    ref = oz.forward(cfg.raw, W, toks)[0]
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    sess = model.init_states(1, 16)
    for sizes in ([300], [1], [5, 40, 2]):
        assert rel(run(sess, toks, sizes), ref) < (1e-4 if fp32 else 1e-3), sizes
    sess.close(); model.close()


def router_margin(cfg, W, token):
    x = W["embed"][token].astype(np.float64) * cfg.raw["embedding"]["scale"]
    z = np.sort(W["l0.mlp.router"] @ (oz.rms(x, cfg.raw["norm"]["eps"]) * W["l0.norm2"]))[::-1]
    top = cfg.raw["layers"][0]["mlp"]["router"]["top"]
    return z[top - 1] - z[top] if top < len(z) else 1.0


@pytest.mark.parametrize("fp32", [True, False])
@pytest.mark.parametrize("window", [2, 63, 64, 65, 130])
def test_one_key_at_the_window_edge(window, fp32):
    """Every query points at one planted token whose score stands far above the rest: its value shows while it is inside the window
    and not one token later — in a prompt and in decoding, wherever pages begin."""
    D, H, d, r, dv, c = 64, 2, 16, 4, 8, 24
    cfg = zt.config(D, 12, [zt.latent_attention(H, d, r, dv, c, window, scale=1.0)], embed_scale=8.0)
    g = np.random.default_rng(window)
    basis = np.linalg.qr(g.standard_normal((c, c)))[0]
    aim = np.ones(d)
    embed = np.zeros((12, D))
    embed[np.arange(12), np.arange(12)] = 1.0                            # token t is channel t; token 0 is the planted one
    dkv = np.zeros((c + r, D))
    for t in range(12):
        dkv[:c, t] = basis[0] if t == 0 else basis[1 + t]
    q = np.zeros((H, d + r, D))
    q[:, :d, :12] = aim[None, :, None] * 0.125
    uk, uv = np.zeros((H, d, c)), np.zeros((H, dv, c))
    uk[:] = 0.2 * np.outer(aim, basis[0])
    uv[:] = np.outer(np.ones(dv), basis[0])
    o = np.zeros((D, H * dv))
    o[50] = 1.0
    tens = replace(list(zt.iter_tensors(cfg, seed=1)), embed=embed, l0__mix__dkv=dkv, l0__mix__q=q, l0__mix__uk=uk, l0__mix__uv=uv, l0__mix__o=o,
                   l0__norm1=np.ones(D), l0__mix__dkv__norm=np.ones(c))
    at, T = 70, window + 140
    toks = g.integers(1, 12, T).astype(np.uint32)
    toks[at] = 0
    W = weights(tens)
    ref, stream = oz.forward(cfg.raw, W, toks)
    seen = stream[0, :, 50]
    assert seen[at:at + window].min() > 5 and np.abs(seen[:at]).max() < 0.5 and np.abs(seen[at + window:]).max() < 0.5
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    sess = model.init_states(1, T)
    for sizes in ([T], [1], [at + window - 1, 1, 1, 50], [at + window, 2], [at + 1, 20, 3]):
        assert rel(run(sess, toks, sizes), ref) < TOL[fp32], sizes
    sess.close(); model.close()


@pytest.mark.parametrize("kind", ["retention", "rglru"])
def test_far_write_survives_in_the_state(kind):
    """Decays near one carry a single early token for hundreds of tokens: changing that token changes late logits by as much as the
    plain implementation says, in prompts and portions."""
    layer = zt.retention(2, 32, 32, [0.9995, 1.0], rot_dims=0) if kind == "retention" else zt.rglru(64, 2)
    cfg = zt.config(64, 60, [layer], embed_scale=2.0)
    tens = list(zt.iter_tensors(cfg, seed=4))
    if kind == "rglru":
        tens = replace(tens, l0__mix__lam=np.full(64, -9.0))
    W = weights(tens)
    toks = np.random.default_rng(2).integers(0, 60, 500).astype(np.uint32)
    toks2 = toks.copy()
    toks2[5] = (toks2[5] + 17) % 60
    want = oz.forward(cfg.raw, W, toks2)[0][-1] - oz.forward(cfg.raw, W, toks)[0][-1]
    assert np.abs(want).max() > 1e-3
    for fp32 in (True, False):
        model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
        sess = model.init_states(1, 16)
        for sizes in ([500], [400, 1, 99]):
            got = run(sess, toks2, sizes)[-1].astype(np.float64) - run(sess, toks, sizes)[-1]
            assert np.abs(got - want).max() < (0.01 if fp32 else 0.1) * np.abs(want).max() + (1e-5 if fp32 else 1e-3)
        sess.close(); model.close()


def test_first_tokens():
    """Sequences of one and two tokens: nothing ahead of position 0 is read (slots used before hold other sequences' inputs)."""
    cfg, tens, W, toks, _ = setup("mixed")
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=True)
    sess = model.init_states(1, 400)
    for T in (1, 2, 3):
        run(sess, toks[100:300], [200])
        assert rel(run(sess, toks[:T], [T]), oz.forward(cfg.raw, W, toks[:T])[0]) < TOL[True]
        run(sess, toks[100:300], [200])
        assert rel(run(sess, toks[:T], [1]), oz.forward(cfg.raw, W, toks[:T])[0]) < TOL[True]
    sess.close(); model.close()


# ---- whole models ----------------------------------------------------------------------------------------------------
def models():
    mixed = [zt.retention(3, 24, 36, [0.9, 0.97, 0.999], rot_dims=16, mlp=zt.moe(7, 3, 24)), zt.rglru(88, 4, conv=3, mlp=zt.dense(72)),
             zt.latent_attention(5, 20, 12, 28, 40, 37, base=500.0, mlp=zt.dense(90))]
    mixed += [zt.again(mixed, 0), zt.rglru(60, 5, conv=2, mlp=zt.moe(4, 1, 40)), zt.again(mixed, 2), zt.again(mixed, 1)]
    mixed.append(zt.latent_attention(2, 16, 8, 16, 64, 70))
    mixed.append(zt.again(mixed + [None], 3))                            # weights of a layer that uses another one's
    return {
        "mixed": zt.config(104, 211, mixed, eps=2e-5, embed_scale=4.0),
        "recurrent": zt.config(64, 97, [zt.retention(2, 64, 64, mlp=zt.dense(64)), zt.rglru(96, 2, mlp=zt.dense(40))], embed_scale=2.0),
        "attention": zt.config(192, 300, [zt.latent_attention(3, 64, 32, 48, 128, 50, mlp=zt.dense(128)), zt.latent_attention(2, 48, 16, 32, 64, 129)]),
    }


_cache = {}


def setup(name, seed=11):
    if name not in _cache:
        cfg = models()[name]
        tens = list(zt.iter_tensors(cfg, seed=seed))
        W = weights(tens)
        toks = np.random.default_rng(seed).integers(0, cfg.vocab_size, 330).astype(np.uint32)
        _cache[name] = (cfg, tens, W, toks, oz.forward(cfg.raw, W, toks)[0])
    return _cache[name]


def close_enough(got, ref, fp32):
    """bf16 through layers that choose experts: where a choice is close the rounding may turn it over, for a few tokens."""
    e = np.abs(np.asarray(got, np.float64) - ref).max(axis=1) / np.sqrt((ref ** 2).mean())
    return e.max() < TOL[fp32] if fp32 else (np.median(e) < TOL[fp32] and (e > 2 * TOL[fp32]).mean() < 0.1)


@pytest.mark.parametrize("fp32", [True, False])
@pytest.mark.parametrize("name", sorted(models()))
def test_model_whole_portions_decode(name, fp32):
    """The whole prompt in one call, portions down to two tokens, and token by token, in slots other than the first too."""
    cfg, tens, W, toks, ref = setup(name)
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    sess = model.init_states(3, 400)
    for slot, sizes in ((0, [330]), (2, [37, 2, 3, 64, 2, 17]), (0, [1]), (1, [300] + [1] * 30)):
        got = run(sess, toks, sizes, slot)
        assert close_enough(got, ref, fp32), (slot, sizes, rel(got, ref))
    # only some places wanted, and none
    sess.reset([1])
    assert sess.extend(toks[:100], [], slot=1).shape[0] == 0
    got = sess.extend(toks[100:200], [0, 7, 99], slot=1)
    assert rel(got, ref[[100, 107, 199]]) < TOL[fp32] * (1 if fp32 else 3)
    sess.close(); model.close()


@pytest.mark.parametrize("fp32", [True, False])
def test_layers_one_by_one(fp32):
    """Every layer fed with the plain implementation's stream; few rows, rows enough for the tensor cores, and for decode steps in
    which the gated recurrence goes by rows of products."""
    cfg, tens, W, toks, _ = setup("mixed")
    stream = oz.forward(cfg.raw, W, toks[:24])[1]
    x0 = W["embed"].astype(np.float64)[toks[:24]] * cfg.raw["embedding"]["scale"]
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    for copies in (1, 12, 40):
        sess = model.init_states(copies, 64)
        for t in range(24):
            x = x0[t]
            for layer in range(cfg.n_layers):
                got = sess.run_block(layer, np.repeat(x[None].astype(np.float32), copies, axis=0))
                x = stream[layer, t]
                assert rel(got, np.repeat(x[None], copies, axis=0)) < TOL[fp32], (copies, t, layer)
        sess.close()
    model.close()


@pytest.mark.parametrize("fp32", [True, False])
@pytest.mark.parametrize("name", sorted(models()))
def test_unequal_prompts_in_a_batch(name, fp32):
    """Prompts of different lengths together (fewer than the tensor-core rows, and more), then decoding together."""
    cfg, tens, W, toks, _ = setup(name)
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    g = np.random.default_rng(3)
    for batch in (3, 11, 40):
        lens = np.concatenate([[1, 200], g.integers(1, 200, batch - 2)]).astype(np.int32)
        prompts = g.integers(0, cfg.vocab_size, (batch, 200 + 6)).astype(np.uint32)
        sess = model.init_states(batch, 256)
        for chunked in (128, 0):            # in slices, and position by position
            sess.reset()
            sess.set_option("chunked_prefill", chunked)
            outs = [sess.prefill_ragged(prompts[:, :200], lens)]
            for i in range(5):
                outs.append(sess.forward_step(prompts[np.arange(batch), lens + i])[0])
            for b in sorted({0, 1, batch - 1}):
                ref = oz.forward(cfg.raw, W, prompts[b, :lens[b] + 5])[0][lens[b] - 1:]
                got = np.stack([o[b] for o in outs])
                assert rel(got, ref) < TOL[fp32] * (1 if fp32 else 2), (batch, chunked, b, rel(got, ref))
        sess.close()
    model.close()


def test_slots_are_used_again():
    """Sequences come and go in the same slots, interleaved with others; nothing of an earlier one is left."""
    cfg, tens, W, _, _ = setup("mixed")
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=True)
    sess = model.init_states(2, 320)
    g = np.random.default_rng(8)
    seqs = [g.integers(0, cfg.vocab_size, n).astype(np.uint32) for n in (300, 5, 120, 2, 81)]
    refs = [oz.forward(cfg.raw, W, t)[0] for t in seqs]
    other = g.integers(0, cfg.vocab_size, 200).astype(np.uint32)
    oref, at = oz.forward(cfg.raw, W, other)[0], 0
    for t, r in zip(seqs, refs):
        sess.reset([1])
        got = []
        for a, n in cuts(len(t), [60, 1, 2]):
            got.append(sess.extend(t[a:a + n], range(n), slot=1))
            if at < 200:
                assert rel(sess.extend(other[at:at + 7], range(min(7, 200 - at)), slot=0), oref[at:at + 7]) < TOL[True]
                at += 7
        assert rel(np.concatenate(got), r) < TOL[True]
    # a snapshot taken in the middle resumes in another slot
    sess.reset()
    sess.extend(seqs[0][:150], [], slot=0)
    snap = sess.save_state(0)
    sess.extend(seqs[0][150:170], [], slot=0)
    sess.load_state(1, snap)
    assert rel(sess.extend(seqs[0][150:], range(150), slot=1), refs[0][150:]) < TOL[True]
    sess.close(); model.close()


@pytest.mark.parametrize("fp32", [True, False])
def test_long_decoding_and_ring_wrap(fp32):
    """Decoding far past the ring, teacher forced, against the whole sequence at once."""
    cfg = zt.config(64, 80, [zt.latent_attention(2, 24, 8, 32, 32, 40, base=100.0, mlp=zt.dense(64)), zt.retention(2, 32, 32), zt.rglru(64, 4)],
                    embed_scale=4.0)
    tens = list(zt.iter_tensors(cfg, seed=2))
    toks = np.random.default_rng(1).integers(0, 80, 700).astype(np.uint32)
    ref = oz.forward(cfg.raw, weights(tens), toks)[0]
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    sess = model.init_states(1, 64)         # ring of 128 tokens: wraps five times
    got = [sess.extend(toks[:150], [0, 149])]
    got += [sess.extend(toks[t:t + 1], [0]) for t in range(150, 700)]
    assert rel(np.concatenate(got), ref[[0] + list(range(149, 700))]) < TOL[fp32]
    sess.close(); model.close()


def test_long_context_is_split_over_ctas():
    """One sequence at a long context without a window: the slices of the context are merged in order; a far key stands out."""
    cfg = zt.config(64, 50, [zt.latent_attention(3, 32, 16, 24, 64, 0)], embed_scale=3.0)
    tens = list(zt.iter_tensors(cfg, seed=6))
    toks = np.random.default_rng(4).integers(0, 50, 1500).astype(np.uint32)
    ref = oz.forward(cfg.raw, weights(tens), toks)[0]
    model = lumi_b200.NmModel.from_tensors(cfg, tens)
    sess = model.init_states(1, 1600)
    got = [sess.extend(toks[:1490], [1489])] + [sess.extend(toks[t:t + 1], [0]) for t in range(1490, 1500)]
    assert rel(np.concatenate(got), ref[1489:]) < 1e-2
    sess.close(); model.close()


@pytest.mark.parametrize("batch", [1, 4, 12])
@pytest.mark.parametrize("fp32", [True, False])
def test_greedy_generation(fp32, batch):
    """Session.generate (prompt in slices, captured decode steps) against greedy decoding of the plain implementation."""
    cfg, tens, W, _, _ = setup("mixed")
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    sess = model.init_states(batch, 128)
    prompts = np.random.default_rng(6).integers(0, cfg.vocab_size, (batch, 40)).astype(np.uint32)
    out, lens, dump, st = sess.generate(prompts, 24, ignore_eos=True, dump_logits=True)
    assert st.kernel_launches > 0 and list(lens) == [24] * batch
    for b in sorted({0, batch - 1}):
        ref = oz.forward(cfg.raw, W, np.concatenate([prompts[b], out[b][:-1]]))[0][39:]      # along the generated tokens
        assert close_enough(dump[:, b], ref, fp32)
        if fp32:
            for i in range(24):
                top = np.sort(ref[i])[-2:]
                assert out[b, i] == np.argmax(ref[i]) or top[1] - top[0] < TOL[fp32] * np.sqrt((ref ** 2).mean())
    if fp32:
        want, margins = oz.greedy(cfg.raw, W, prompts[0], 10)
        assert min(margins) < 1e-4 or list(out[0][:10]) == want
    # the same tokens without the dump (the fused greedy head where it applies) and by single steps
    sess.reset()
    again = sess.generate(prompts, 24, ignore_eos=True)[0]
    assert np.array_equal(again, out)
    sess.close(); model.close()


def test_score_and_large_vocabulary():
    """Teacher-forced log-probabilities, and the fused greedy head (vocabularies from 4096) with a padded width and a head that is not
    the embedding."""
    cfg = zt.config(72, 5000, [zt.retention(2, 16, 16), zt.latent_attention(2, 16, 8, 16, 32, 30, mlp=zt.dense(32))], embed_scale=4.0)
    tens = list(zt.iter_tensors(cfg, seed=7))
    W = weights(tens)
    model = lumi_b200.NmModel.from_tensors(cfg, tens)
    sess = model.init_states(2, 256)
    toks = np.random.default_rng(3).integers(0, 5000, (2, 150)).astype(np.uint32)
    got = sess.score(toks)
    for b in range(2):
        lg = oz.forward(cfg.raw, W, toks[b])[0]
        lp = lg - np.log(np.sum(np.exp(lg - lg.max(1, keepdims=True)), axis=1, keepdims=True)) - lg.max(1, keepdims=True)
        assert np.abs(got[b] - lp[np.arange(149), toks[b, 1:]]).max() < 5e-2
    sess.reset()
    a = sess.generate(toks[:, :20], 12, ignore_eos=True, dump_logits=True)[0]
    sess.reset()
    assert np.array_equal(a, sess.generate(toks[:, :20], 12, ignore_eos=True)[0])
    sess.close(); model.close()


def test_a_row_does_not_depend_on_the_batch():
    """Decode steps of the same sequence alone, among few and among many others (every form of the kernels), bf16."""
    cfg, tens, W, toks, ref = setup("recurrent")
    model = lumi_b200.NmModel.from_tensors(cfg, tens)
    outs = []
    for batch in (1, 7, 20, 70):
        sess = model.init_states(batch, 128)
        prompts = np.random.default_rng(batch).integers(0, cfg.vocab_size, (batch, 60)).astype(np.uint32)
        prompts[batch // 2] = toks[:60]
        sess.prefill(prompts[:, :50])
        outs.append(np.stack([sess.forward_step(prompts[:, t])[0][batch // 2] for t in range(50, 60)]))
        sess.close()
    for o in outs:
        assert rel(o, ref[50:60]) < 2e-3
    model.close()


@pytest.mark.parametrize("fp32", [True, False])
def test_many_sequences_in_short_slices(fp32):
    """More heads than the GPU holds at a time, several tokens per slice without the chunked form, equal and unequal lengths."""
    cfg, tens, W, _, _ = setup("recurrent")
    batch = 200
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    sess = model.init_states(batch, 64)
    g = np.random.default_rng(5)
    prompts = g.integers(0, cfg.vocab_size, (batch, 14)).astype(np.uint32)
    lens = g.integers(1, 10, batch).astype(np.int32)
    lens[:2] = 9, 1
    for ragged in (False, True):
        sess.reset()
        n = lens if ragged else np.full(batch, 9, np.int32)
        outs = [sess.prefill_ragged(prompts[:, :9], n) if ragged else sess.prefill(prompts[:, :9])]
        for i in range(4):
            outs.append(sess.forward_step(prompts[np.arange(batch), n + i])[0])
        for b in (0, 1, 77, 199):
            ref = oz.forward(cfg.raw, W, prompts[b, :n[b] + 4])[0][n[b] - 1:]
            assert rel(np.stack([o[b] for o in outs]), ref) < (1e-4 if fp32 else 2e-3), (ragged, b)
    sess.close(); model.close()


def test_cache_capacity_is_reported():
    """A cache smaller than the window refuses positions it cannot hold."""
    cfg = zt.config(64, 50, [zt.latent_attention(2, 16, 8, 16, 32, 100)])
    model = lumi_b200.NmModel.from_tensors(cfg, zt.iter_tensors(cfg))
    sess = model.init_states(1, 30)
    sess.extend(np.zeros(30, np.uint32), [29])
    with pytest.raises(lumi_b200.LumiError) as e:
        sess.extend(np.zeros(1, np.uint32), [0])
    assert e.value.code == -9
    sess.close(); model.close()


def test_command_lines(tmp_path):
    """The generate command and the trace replay on a model folder, against the session API."""
    cfg, tens, W, toks, ref = setup("mixed")
    cpath, mpath = zt.write_model_dir(str(tmp_path / "m"), cfg, seed=11)
    cli = os.path.join(os.path.dirname(lumi_b200.LIB_PATH), "lumi-infer-b200")
    ids = [int(t) for t in toks[:12]]
    run_ = subprocess.run([cli, "generate", "-m", mpath, "-c", cpath, "--prompt-ids", ",".join(map(str, ids)), "--max-tokens", "9",
                           "--temperature", "0", "--ignore-eos"], capture_output=True, timeout=300)
    assert run_.returncode == 0, run_.stderr.decode()
    model = lumi_b200.NmModel.load(mpath, cpath)
    sess = model.init_states(1, 64)
    out = sess.generate(np.array([ids], np.uint32), 9, ignore_eos=True)[0][0]
    assert [int(t) for t in run_.stdout.split()] == [int(t) for t in out]
    sess.close(); model.close()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [int(t) for t in toks[:50]], "want": [49, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [1, 2], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [int(toks[50])], "want": [0]}], "end": ["a"]}]
    for dtype, fp32 in (("bfloat16", False), ("float32", True)):
        o = tmp_path / dtype
        o.mkdir()
        run_ = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(o), "--max-tokens", "64"],
                              input="".join(json.dumps(s) + "\n" for s in steps).encode(), capture_output=True, timeout=300)
        assert run_.returncode == 0, run_.stderr.decode()
        assert run_.stdout.decode().split("\n")[:3] == ["done 0", "done 1", "done 2"]
        got = np.concatenate([np.fromfile(o / f, "<f4").reshape(-1, cfg.vocab_size) for f in ("0.f32", "2.f32")])
        assert not (o / "1.f32").exists()
        assert rel(got, ref[[49, 3, 50]]) < TOL[fp32]
