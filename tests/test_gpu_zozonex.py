"""GPU: the Zozonex design — each mechanism alone, then whole models through the session API — against the plain
implementation in oracle/zozonex.py."""
import json
import os
import subprocess

import numpy as np
import pytest

import lumi_b200
from lumi_b200 import synth, zozonex as zz
from oracle import zozonex as oz

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _torch():
    import torch
    return torch


def dev(a, dtype=np.float32):
    return _torch().from_numpy(np.ascontiguousarray(a, dtype=dtype)).cuda()


def rel(got, ref):
    """Error of rows relative to the reference's root mean square."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    return float(np.abs(got - ref).max() / np.sqrt((ref ** 2).mean()))


def call(name, *args):
    lumi_b200.api.check(getattr(lumi_b200.lib(), name)(*args))


def cuts(T, sizes):
    out, at = [], 0
    while at < T:
        n = min(sizes[len(out) % len(sizes)], T - at)
        out.append((at, n))
        at += n
    return out


# ---- the delta rule alone ------------------------------------------------------------------------------------
DELTA_SIZES = [  # heads, kv_heads, dk, dv, taps
    (4, 2, 64, 64, 4), (3, 3, 20, 48, 3), (6, 2, 96, 80, 1), (2, 1, 128, 128, 5), (5, 1, 16, 8, 2), (1, 1, 250, 40, 4), (2, 2, 33, 130, 2)]


def delta_case(H, G, dk, dv, taps, nseq, T, seed):
    g = np.random.default_rng(seed)
    parts = [G * dk, G * dk, H * dv, H, H, H * dv]
    off = np.cumsum([0] + [(p + 7) // 8 * 8 for p in parts])
    ldp = int(off[-1])
    proj = g.standard_normal((nseq, T, ldp))
    conv = [0.7 * g.standard_normal((n, taps)) for n in parts[:3]]
    a_log, dt_bias = g.uniform(-3, 4, H), g.uniform(-4, 3, H)
    return proj.astype(np.float32), off[:6].astype(np.int32), [c.astype(np.float32) for c in conv], a_log.astype(np.float32), \
        dt_bias.astype(np.float32), (1 + 0.3 * g.standard_normal(dv)).astype(np.float32)


def delta_reference(proj, off, conv, a_log, dt_bias, o_norm, H, G, dk, dv, eps):
    outs, states = [], []
    for p in proj.astype(np.float64):
        T = p.shape[0]
        take = lambda i, n: p[:, off[i]:off[i] + n]
        q = oz.silu(oz.short_conv(take(0, G * dk), conv[0])).reshape(T, G, dk)
        k = oz.silu(oz.short_conv(take(1, G * dk), conv[1])).reshape(T, G, dk)
        v = oz.silu(oz.short_conv(take(2, H * dv), conv[2])).reshape(T, H, dv)
        q, k = oz.unit(q) * dk ** -0.5, oz.unit(k)
        beta, dec = oz.sigmoid(take(3, H)), oz.delta_decay(take(4, H), a_log.astype(np.float64), dt_bias.astype(np.float64))
        o, S = np.zeros((T, H, dv)), []
        for h in range(H):
            o[:, h], s = oz.delta_rule(q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], dec[:, h], beta[:, h])
            S.append(s)
        outs.append(oz.gated_head_norm(o, take(5, H * dv).reshape(T, H, dv), o_norm, eps).reshape(T, H * dv))
        states.append(S)
    return np.stack(outs), np.array(states)


@pytest.mark.parametrize("H,G,dk,dv,taps", DELTA_SIZES)
@pytest.mark.parametrize("sizes", [[1], [150], [64, 2, 37, 1, 1, 16], [2, 3]])
def test_delta_rule_alone(H, G, dk, dv, taps, sizes):
    """Token by token, and in chunks wherever a portion has several tokens; portions end anywhere in a chunk."""
    torch = _torch()
    nseq, T, eps = 2, 150, 1e-4
    proj, off, conv, a_log, dt_bias, o_norm = delta_case(H, G, dk, dv, taps, nseq, T, H * 100 + dk)
    ref, Sref = delta_reference(proj, off, conv, a_log, dt_bias, o_norm, H, G, dk, dv, eps)
    dvp, dk4 = (dv + 3) // 4 * 4, (dk + 3) // 4 * 4
    w = [dev(x) for x in conv + [a_log, dt_bias, o_norm]]
    for chunked in (0, 1):
        S = torch.zeros((nseq, H, dk, dvp), device="cuda")
        ring = torch.full((nseq, taps, 2 * G * dk + H * dv), float("nan"), device="cuda")      # nothing ahead of position 0 is read
        scratch = torch.empty(nseq * T * (2 * G * dk4 + 2 * H * dvp + 2 * H), device="cuda")
        got = np.zeros_like(ref)
        for at, n in cuts(T, sizes):
            rows = dev(proj[:, at:at + n].reshape(nseq * n, -1))
            pos = dev([at] * nseq, np.int32)
            y = torch.empty((nseq, n, H * dv), device="cuda")
            torch.cuda.synchronize()
            call("lumi_k_delta_rule", rows.data_ptr(), proj.shape[2], off.ctypes.data, *[x.data_ptr() for x in w], S.data_ptr(), ring.data_ptr(),
                 pos.data_ptr(), y.data_ptr(), scratch.data_ptr(), H, G, dk, dv, taps, eps, nseq, n, int(chunked and n > 1), 0)
            torch.cuda.synchronize()
            got[:, at:at + n] = y.cpu().numpy()
        # a read-out near zero is normalised up: compare against each head's own scale
        assert rel(got, ref) < 2e-3 and np.sqrt(np.mean((got - ref) ** 2) / np.mean(ref ** 2)) < 2e-5, chunked
        assert rel(S.cpu().numpy()[..., :dv], Sref) < 1e-4


# ---- attention alone -------------------------------------------------------------------------------------------
ATT_SIZES = [  # heads, kv_heads, dk, dv, window
    (4, 4, 64, 64, 100), (6, 2, 80, 48, 33), (8, 1, 32, 96, 1), (20, 1, 24, 40, 64), (3, 3, 100, 20, 65), (4, 2, 128, 128, 200), (2, 1, 192, 256, 50),
    (4, 4, 64, 64, 0)]


def paged(nseq, pages, torch, seed):
    """Pages of all sequences in one shuffled pool."""
    perm = np.random.default_rng(seed).permutation(nseq * pages).astype(np.int32)
    return torch.from_numpy(perm.reshape(nseq, pages)).cuda()


def run_attention(proj, off, H, G, dk, dv, window, scale, sizes, bf16, pages, qk_norm=1, sink=1, eps=1e-5):
    torch = _torch()
    nseq, T, ldp = proj.shape
    esz = torch.bfloat16 if bf16 else torch.float32
    r16 = lambda n: (n + 15) // 16 * 16
    kv = torch.full((nseq * pages, G, 64 * (r16(dk) + r16(dv))), float("nan"), dtype=esz, device="cuda")      # unused slots must not matter
    table = paged(nseq, pages, torch, T + dk)
    got = np.zeros((nseq, T, H * dv), np.float32)
    for at, n in cuts(T, sizes):
        rows, pos = dev(proj[:, at:at + n].reshape(nseq * n, -1)), dev([at] * nseq, np.int32)
        y = torch.empty((nseq, n, H * dv), device="cuda")
        torch.cuda.synchronize()
        call("lumi_k_window_attention", rows.data_ptr(), ldp, off.ctypes.data, kv.data_ptr(), 1 if bf16 else 0, table.data_ptr(), pages,
             pos.data_ptr(), y.data_ptr(), H, G, dk, dv, window, scale, qk_norm, sink, eps, 1, nseq, n, 0)
        torch.cuda.synchronize()
        got[:, at:at + n] = y.cpu().numpy()
    return got


def attention_reference(proj, off, H, G, dk, dv, window, scale, qk_norm=True, sink=True, eps=1e-5, bf16=False):
    """bf16: keys and values as a bf16 cache holds them."""
    held = (lambda x: synth.bf16_bits_to_f32(synth.f32_to_bf16_bits(x)).astype(np.float64)) if bf16 else (lambda x: x)
    out = []
    for p in proj.astype(np.float64):
        T = p.shape[0]
        q = p[:, off[0]:off[0] + H * dk].reshape(T, H, dk)
        k = p[:, off[1]:off[1] + G * dk].reshape(T, G, dk)
        v = p[:, off[2]:off[2] + G * dv].reshape(T, G, dv)
        if qk_norm:
            q, k = oz.rms(q, eps), oz.rms(k, eps)
        k, v = held(k), held(v)
        if sink:
            out.append(oz.attention(q, k, v, scale, window).reshape(T, H * dv))
        else:
            o = np.zeros((T, H, dv))
            mask = oz.window_mask(T, window)
            for h in range(H):
                s = np.where(mask, q[:, h] @ k[:, h // (H // G)].T * scale, -np.inf)
                e = np.exp(s - s.max(1, keepdims=True))
                o[:, h] = e / e.sum(1, keepdims=True) @ v[:, h // (H // G)]
            out.append(o.reshape(T, H * dv))
    return np.stack(out)


def attention_rows(nseq, T, H, G, dk, dv, seed):
    g = np.random.default_rng(seed)
    off = np.array([0, H * dk, H * dk + G * dk], np.int32)
    return g.standard_normal((nseq, T, H * dk + G * (dk + dv))).astype(np.float32), off


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("H,G,dk,dv,window", ATT_SIZES)
def test_attention_alone(H, G, dk, dv, window, bf16):
    """Whole prompt, single tokens and uneven portions through a ring that wraps several times; with and without the sink and the
    norm of q and k."""
    T = 230
    proj, off = attention_rows(2, T, H, G, dk, dv, dk + dv)
    scale = 1.7 * dk ** -0.5
    tol = 4e-3 if bf16 else 2e-5            # (a key on a rounding border may fall to the other side)
    whole_pages = (max(window, 1) + T - 1 + 63) // 64 if window else (T + 63) // 64
    small_pages = (max(window, 1) + 70 - 1 + 63) // 64 if window else whole_pages
    ref = attention_reference(proj, off, H, G, dk, dv, window, scale, bf16=bf16)
    for sizes, pages in (([T], whole_pages), ([1], small_pages), ([70, 2, 3, 1, 41], small_pages)):
        got = run_attention(proj, off, H, G, dk, dv, window, scale, sizes, bf16, pages)
        assert rel(got, ref) < tol, (sizes, rel(got, ref))
    ref = attention_reference(proj, off, H, G, dk, dv, window, scale, qk_norm=False, sink=False, bf16=bf16)
    got = run_attention(proj, off, H, G, dk, dv, window, scale, [100, 1, 1, 28], bf16, whole_pages, qk_norm=0, sink=0)
    assert rel(got, ref) < tol


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("window", [2, 63, 64, 65, 130])
def test_one_key_at_the_window_edge(window, bf16):
    """Every query points at one planted key whose score stands far above the rest: the context is that key's value while the key
    is inside the window, and nothing of it one token later — in a prompt and in decoding, wherever pages begin."""
    H, G, dk, dv = 2, 1, 32, 32
    T, at = window + 140, 70
    proj, off = attention_rows(1, T, H, G, dk, dv, window)
    aim = np.random.default_rng(5).standard_normal(dk).astype(np.float32)
    proj[:, :, :H * dk] = np.tile(aim, H)                               # all queries
    keys = proj[:, :, off[1]:off[1] + dk]
    keys -= (keys @ aim / (aim @ aim))[..., None] * aim                  # other keys: score 0
    keys[:, at] = aim
    proj[:, at, off[2]:] = 40.0
    scale = 12.0 / dk
    ref = attention_reference(proj, off, H, G, dk, dv, window, scale)
    assert ref[0, at + window - 1].min() > 30 and np.abs(ref[0, at + window]).max() < 5
    for sizes in ([T], [1], [at + window - 1, 1, 1, 50], [at + window, 2]):
        pages = (window + max(sizes) + 63) // 64
        got = run_attention(proj, off, H, G, dk, dv, window, scale, sizes, bf16, pages)
        assert np.abs(got - ref).max() < (0.3 if bf16 else 1e-3), sizes


def test_sink_takes_the_weight_when_nothing_matches():
    """Scores far below zero: almost all weight goes to the sink and the context vanishes; one token alone keeps 1 / (1 + e^-s)."""
    H, G, dk, dv = 1, 1, 16, 16
    proj, off = attention_rows(1, 8, H, G, dk, dv, 3)
    proj[:, :, off[1]:off[1] + dk] = -proj[:, :, :dk]                    # key = -query
    for bf16 in (False, True):
        got = run_attention(proj, off, H, G, dk, dv, 1, 1.0, [8], bf16, 1)
        ref = proj[:, :, off[2]:] / (1 + np.exp(16.0))
        assert np.abs(got - ref).max() < 1e-8


def test_context_split_over_ctas_and_all_keys():
    """One sequence decoding at a long context: the slices of the context are merged in order."""
    H, G, dk, dv, T = 4, 2, 64, 64, 1500
    proj, off = attention_rows(1, T, H, G, dk, dv, 9)
    proj[:, 3, off[1]:off[1] + G * dk] = np.tile(proj[0, T - 1, :dk], G)      # a far key that the last query looks for
    for window in (0, 1200):
        ref = attention_reference(proj, off, H, G, dk, dv, window, 0.4, bf16=True)
        got = run_attention(proj, off, H, G, dk, dv, window, 0.4, [T - 3, 1], True, (T + max(window, 1) + 63) // 64)
        assert rel(got[:, -3:], ref[:, -3:]) < 2e-3


# ---- norm into the residual stream alone -----------------------------------------------------------------------
@pytest.mark.parametrize("width", [40, 64, 1000, 5000])
def test_norm_add_alone(width):
    torch = _torch()
    ld = (width + 63) // 64 * 64
    g = np.random.default_rng(width)
    pad = lambda a: np.pad(a, [(0, 0)] * (a.ndim - 1) + [(0, ld - width)])
    x, o, w = g.standard_normal((5, width)), 1e-3 * g.standard_normal((5, width)), 1 + 0.2 * g.standard_normal(width)
    xd, od, wd = dev(pad(x)), dev(pad(o)), dev(pad(w))
    hi, lo = torch.empty((5, ld), dtype=torch.bfloat16, device="cuda"), torch.empty((5, ld), dtype=torch.bfloat16, device="cuda")
    torch.cuda.synchronize()
    call("lumi_k_norm_add", xd.data_ptr(), od.data_ptr(), wd.data_ptr(), 0, hi.data_ptr(), lo.data_ptr(), 5, width, ld, 1e-6, 0)
    y = torch.empty((5, ld), device="cuda")
    call("lumi_k_norm_add", od.data_ptr(), 0, wd.data_ptr(), y.data_ptr(), 0, 0, 5, width, ld, 1e-6, 0)
    torch.cuda.synchronize()
    ref = oz.rms(o, 1e-6) * w
    assert np.abs(xd.cpu().numpy()[:, :width] - (x + ref)).max() < 1e-5
    assert np.abs((hi.float() + lo.float()).cpu().numpy() - xd.cpu().numpy()).max() < 1e-4
    assert np.abs(y.cpu().numpy()[:, :width] - ref).max() < 1e-5
    assert float(xd[:, width:].abs().sum()) == 0 and float(y[:, width:].abs().sum()) == 0


# ---- whole models ----------------------------------------------------------------------------------------------------
def models():
    return {
        # widths and heads off every tile size; more query than key heads; sharing layers with a wider and a narrower window
        "mixed": zz.config(104, 211, [zz.attention(6, 24, 20, vdim=40, kv_heads=2, ff=72), zz.delta(4, 36, 20, kv_heads=2, conv=3, ff=88),
                                      zz.attention(6, 24, 70, vdim=40, kv_heads=2, kv_from=0), zz.delta(3, 16, 48, conv=2),
                                      zz.attention(6, 24, 7, vdim=40, kv_heads=2, ff=40, kv_from=0)], eps=3e-4, embed_scale=5.0),
        "delta_only": zz.config(64, 97, [zz.delta(2, 64, 64, kv_heads=1, ff=64), zz.delta(2, 32, 96, conv=1)], embed_scale=2.0),
        "attention_only": zz.config(192, 300, [zz.attention(3, 64, 50, ff=128), zz.attention(2, 48, 129, vdim=32, kv_heads=1, ff=64)], eps=1e-6),
    }


_cache = {}


def setup(name, seed=11):
    if name not in _cache:
        cfg = models()[name]
        tens = list(zz.iter_tensors(cfg, seed=seed))
        W = {n: synth.as_f32(dt, a) for n, dt, a in tens}
        toks = np.random.default_rng(seed).integers(0, cfg.vocab_size, 330).astype(np.uint32)
        _cache[name] = (cfg, tens, W, toks, oz.forward(cfg.raw, W, toks)[0])
    return _cache[name]


TOL = {True: 1e-4, False: 3e-2}      # fp32 / bf16 weights and cache; worst logit over the logits' root mean square


@pytest.mark.parametrize("fp32", [True, False])
@pytest.mark.parametrize("name", sorted(models()))
def test_model_whole_portions_decode(name, fp32):
    """The whole prompt in one call, portions down to two tokens, and token by token, in slots other than the first too."""
    cfg, tens, W, toks, ref = setup(name)
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    sess = model.init_states(3, 400)
    for slot, sizes in ((0, [330]), (2, [37, 2, 3, 64, 2, 17]), (0, [1]), (1, [300] + [1] * 30)):
        sess.reset([slot])
        got = np.concatenate([sess.extend(toks[at:at + n], range(n), slot=slot) for at, n in cuts(330, sizes)])
        assert rel(got, ref) < TOL[fp32], (slot, sizes, rel(got, ref))
    # only some places wanted, and none
    sess.reset([1])
    assert sess.extend(toks[:100], [], slot=1).shape[0] == 0
    got = sess.extend(toks[100:200], [0, 7, 99], slot=1)
    assert rel(got, ref[[100, 107, 199]]) < TOL[fp32]
    sess.close(); model.close()


@pytest.mark.parametrize("fp32", [True, False])
def test_layers_one_by_one(fp32):
    cfg, tens, W, toks, _ = setup("mixed")
    stream = oz.forward(cfg.raw, W, toks[:30])[1]
    x0 = oz.embed(W["embed"].astype(np.float64), toks[:30], cfg.raw["embedding"]["scale"])
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    for copies in (1, 12):                  # the weight-streaming kernels, then the tensor cores
        sess = model.init_states(copies, 64)
        for t in range(30):
            x = np.repeat(x0[t:t + 1].astype(np.float32), copies, axis=0)
            for layer in range(cfg.n_layers):
                x = sess.run_block(layer, x)
                assert rel(x, np.repeat(stream[layer, t:t + 1], copies, axis=0)) < TOL[fp32], (copies, t, layer)
        sess.close()
    model.close()


@pytest.mark.parametrize("fp32", [True, False])
@pytest.mark.parametrize("name", sorted(models()))
def test_unequal_prompts_in_a_batch(name, fp32):
    """Prompts of different lengths together (fewer than the tensor-core rows, and more), then decoding together."""
    cfg, tens, W, toks, _ = setup(name)
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    g = np.random.default_rng(3)
    for batch in (3, 11):
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
                assert rel(got, ref) < TOL[fp32], (batch, chunked, b, rel(got, ref))
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
    cfg = zz.config(64, 80, [zz.attention(2, 32, 40, ff=64), zz.delta(2, 32, 32), zz.attention(2, 32, 25, kv_from=0)], embed_scale=4.0)
    tens = list(zz.iter_tensors(cfg, seed=2))
    W = {n: synth.as_f32(dt, a) for n, dt, a in tens}
    toks = np.random.default_rng(1).integers(0, 80, 700).astype(np.uint32)
    ref = oz.forward(cfg.raw, W, toks)[0]
    model = lumi_b200.NmModel.from_tensors(cfg, tens, widen_weights=fp32)
    sess = model.init_states(1, 64)         # ring of 128 tokens: wraps five times
    got = [sess.extend(toks[:150], [0, 149])]
    got += [sess.extend(toks[t:t + 1], [0]) for t in range(150, 700)]
    assert rel(np.concatenate(got), ref[[0] + list(range(149, 700))]) < TOL[fp32]
    sess.close(); model.close()


def test_far_write_survives_in_the_state():
    """A delta-rule layer whose decays are near one carries a single early token for hundreds of tokens: changing that token
    changes late logits by as much as the plain implementation says, in the chunked form too."""
    cfg = zz.config(64, 60, [zz.delta(2, 32, 32, kv_heads=1)], embed_scale=2.0)
    tens = [(n, dt, (synth.f32_to_bf16_bits(np.full(a.shape, -8.0, np.float32)) if n.endswith(("A_log", "dt_bias")) else a))
            for n, dt, a in zz.iter_tensors(cfg, seed=4)]
    W = {n: synth.as_f32(dt, a) for n, dt, a in tens}
    toks = np.random.default_rng(2).integers(0, 60, 400).astype(np.uint32)
    toks2 = toks.copy()
    toks2[5] = (toks2[5] + 17) % 60
    want = oz.forward(cfg.raw, W, toks2)[0][-1] - oz.forward(cfg.raw, W, toks)[0][-1]
    model = lumi_b200.NmModel.from_tensors(cfg, tens)
    sess = model.init_states(2, 400)
    got = sess.extend(toks2, [399], slot=1)[0].astype(np.float64) - sess.extend(toks, [399], slot=0)[0]
    assert np.abs(want).max() > 1e-3
    assert np.abs(got - want).max() < 0.15 * np.abs(want).max() + 2e-3
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
        assert rel(dump[:, b], ref) < TOL[fp32]
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
    """Teacher-forced log-probabilities, and the fused greedy head (vocabularies from 4096) with a padded width."""
    cfg = zz.config(72, 5000, [zz.delta(2, 16, 16), zz.attention(2, 16, 30, ff=32)], embed_scale=4.0)
    tens = list(zz.iter_tensors(cfg, seed=7))
    W = {n: synth.as_f32(dt, a) for n, dt, a in tens}
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


def test_cache_capacity_is_reported():
    """A cache smaller than the window refuses positions it cannot hold."""
    cfg = zz.config(64, 50, [zz.attention(2, 16, 100)])
    model = lumi_b200.NmModel.from_tensors(cfg, zz.iter_tensors(cfg))
    sess = model.init_states(1, 30)
    sess.extend(np.zeros(30, np.uint32), [29])
    with pytest.raises(lumi_b200.LumiError) as e:
        sess.extend(np.zeros(1, np.uint32), [0])
    assert e.value.code == -9
    sess.close(); model.close()


def test_command_lines(tmp_path):
    """The generate command and the trace replay on a model folder, against the session API."""
    cfg, tens, W, toks, ref = setup("mixed")
    cpath, mpath = zz.write_model_dir(str(tmp_path / "m"), cfg, seed=11)
    cli = os.path.join(os.path.dirname(lumi_b200.LIB_PATH), "lumi-infer-b200")
    ids = [int(t) for t in toks[:12]]
    run = subprocess.run([cli, "generate", "-m", mpath, "-c", cpath, "--prompt-ids", ",".join(map(str, ids)), "--max-tokens", "9",
                          "--temperature", "0", "--ignore-eos"], capture_output=True, timeout=300)
    assert run.returncode == 0, run.stderr.decode()
    model = lumi_b200.NmModel.load(mpath, cpath)
    sess = model.init_states(1, 64)
    out = sess.generate(np.array([ids], np.uint32), 9, ignore_eos=True)[0][0]
    assert [int(t) for t in run.stdout.split()] == [int(t) for t in out]
    sess.close(); model.close()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [int(t) for t in toks[:50]], "want": [49, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [1, 2], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [int(toks[50])], "want": [0]}], "end": ["a"]}]
    for dtype, fp32 in (("bfloat16", False), ("float32", True)):
        o = tmp_path / dtype
        o.mkdir()
        run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(o), "--max-tokens", "64"],
                             input="".join(json.dumps(s) + "\n" for s in steps).encode(), capture_output=True, timeout=300)
        assert run.returncode == 0, run.stderr.decode()
        assert run.stdout.decode().split("\n")[:3] == ["done 0", "done 1", "done 2"]
        got = np.concatenate([np.fromfile(o / f, "<f4").reshape(-1, cfg.vocab_size) for f in ("0.f32", "2.f32")])
        assert not (o / "1.f32").exists()
        assert rel(got, ref[[49, 3, 50]]) < TOL[fp32]
