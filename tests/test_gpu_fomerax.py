"""GPU tests of the Fomerax architecture: every mechanism's kernel against plain numpy (float64) written from the equations
(oracle/fomerax.py), then the engine — whole prompts, token-by-token decoding, portions down to two tokens, mixed batches
with reused pages, windows that pass over decoded tokens, greedy generation through LLMEngine.generate and a replay through
bin/trace_run — on small random models.  f32 engines must agree with the oracle to rounding; bf16 engines within the error of
bf16 operands.  Where random weights would hide a fault (one key among hundreds, a window's edge, a slope's reach) the inputs
are made so that one score stands out."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import fomerax as F
from tests.arch_util import cut, dev_i, dev_t, engine_on, f32r, npf, paged, rel_err, replay, write_checkpoint

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF16 = torch.float32, torch.bfloat16
DTYPES = [F32, BF16]


def draw(rng, shape, dtype, scale=1.0):
    """Numbers that `dtype` represents exactly, as float64."""
    a = rng.standard_normal(shape) * scale
    return F.bf16_round(a) if dtype == BF16 else f32r(a)


def snap(a, dtype):
    return F.bf16_round(a) if dtype == BF16 else f32r(a)


# ------------------------------------------------------------------------------------------------ mechanisms alone

@pytest.mark.parametrize("dims,base,scaling", [
    (32, 1e4, (4.0, 32.0, 1.0, 512)), (2, 100.0, (3.0, 4.0, 1.0, 60)), (12, 5e4, (16.0, 8.0, 2.0, 4096)), (64, 1e4, (40.0, 32.0, 1.0, 4096)),
    (8, 50.0, (2.0, 1.0, 1.0, 100)),          # both ends at one pair
    (16, 10.0, (5.0, 100.0, 50.0, 30)),       # everything is slower than both: lo and hi below the first pair
    (6, 1e6, (1.0, 2.0, 1.0, 64)),            # factor 1: plain rotary
    (10, 1.5, (7.0, 3.0, 0.001, 1000))])      # hi beyond the last pair
def test_yarn_table(cuda, dims, base, scaling):
    from nano_vllm_rs_b200 import ops
    tab = npf(ops.rope_table_yarn(900, dims, base, *scaling, cuda))
    f, amp = F.yarn_frequencies(base, dims, dict(zip(("factor", "fast", "slow", "original"), scaling)))
    a = np.arange(900)[:, None] * f[None, :]
    np.testing.assert_allclose(tab, np.stack([np.cos(a) * amp, np.sin(a) * amp], -1), atol=2e-6)


def yarn_np(max_pos, dims, base, scaling):
    f, amp = F.yarn_frequencies(base, dims, scaling)
    a = np.arange(max_pos, dtype=np.float64)[:, None] * f[None, :]
    return np.stack([np.cos(a) * amp, np.sin(a) * amp], -1)


YARN = {"factor": 3.0, "fast": 4.0, "slow": 1.0, "original": 60}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("QR,R,rd,dense", [(10, 7, 4, False), (88, 72, 32, True), (1, 1, 2, True), (40, 128, 8, False), (130, 516, 64, True), (12, 20, 6, True),
                                           (8, 24, 0, True)])
def test_latent_rows_are_normed_rotated_and_stored(cuda, dtype, QR, R, rd, dense):
    from nano_vllm_rs_b200 import ops
    rng = np.random.default_rng(QR + R)
    n, eps, rows, max_pos, base = 11, 1e-5, 40, 600, 50.0
    row = (R + rd + 7) // 8 * 8
    off = QR + (4 if QR % 4 == 0 else 3)                               # a gap between the two latents
    ld = (off + R + rd + 5 + 7) // 8 * 8
    proj, pos = f32r(rng.standard_normal((n, ld)) * 2), rng.integers(0, max_pos, n)
    pos[0] = 0
    slots = rng.permutation(rows)[:n].astype(np.int32); slots[4] = -1
    qw, cw = f32r(1 + 0.3 * rng.standard_normal(QR)), f32r(1 + 0.3 * rng.standard_normal(R))
    tab = dev_t(yarn_np(max_pos, rd, base, YARN), cuda) if rd else None
    cache = torch.full((rows, row), 7.0, device=cuda, dtype=dtype)
    dn = torch.full((n, row), 7.0, device=cuda, dtype=dtype) if dense else None
    cq = ops.latent_norm_store(dev_t(proj, cuda), QR, dev_t(qw, cuda), off, R, rd, dev_t(cw, cuda), eps, dev_i(pos, cuda, torch.int64), tab, rd, cache,
                               dev_i(slots, cuda), dtype, dense=dn)
    tol = dict(rtol=2e-5, atol=2e-5) if dtype == F32 else dict(rtol=1e-2, atol=1e-2)
    np.testing.assert_allclose(npf(cq), np.stack([F.rms(proj[t, :QR], eps) * qw for t in range(n)]), **tol)
    ref = np.full((rows, row), 7.0)
    for t in range(n):
        r = np.concatenate([F.rms(proj[t, off:off + R], eps) * cw, F.rotate_pairs(proj[t, off + R:off + R + rd], pos[t], base, YARN) if rd else []])
        if slots[t] >= 0:
            ref[slots[t], :R + rd] = r
        if dense:
            np.testing.assert_allclose(npf(dn)[t, :R + rd], r, **tol)
            assert (npf(dn)[t, R + rd:] == 7.0).all()
    np.testing.assert_allclose(npf(cache), ref, **tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,rd", [(3, 6, 4), (4, 64, 32), (1, 8, 8), (2, 5, 2), (16, 128, 64), (3, 16, 24)])
def test_rotated_part_of_the_queries(cuda, dtype, H, D, rd):
    from nano_vllm_rs_b200 import ops
    rng = np.random.default_rng(H + D)
    n, max_pos, base = 9, 500, 80.0
    x, pos = draw(rng, (n, H, D + rd), dtype), rng.integers(0, max_pos, n)
    xd = dev_t(x.reshape(n, -1), cuda, dtype)
    ops.rotate_tail(xd, dev_i(pos, cuda, torch.int64), dev_t(yarn_np(max_pos, rd, base, YARN), cuda), rd, H, D, rd)
    got = npf(xd).reshape(n, H, D + rd)
    np.testing.assert_array_equal(got[:, :, :D], x[:, :, :D])
    ref = np.stack([[F.rotate_pairs(x[t, h, D:], pos[t], base, YARN) for h in range(H)] for t in range(n)])
    np.testing.assert_allclose(got[:, :, D:], ref, **(dict(rtol=2e-5, atol=2e-5) if dtype == F32 else dict(rtol=1e-2, atol=1e-2)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q,k,v", [(12, 8, 4), (7, 5, 3), (128, 64, 64), (1, 1, 1)])
def test_projection_columns_go_to_queries_and_cache(cuda, dtype, q, k, v):
    from nano_vllm_rs_b200 import ops
    rng = np.random.default_rng(q)
    n, rows = 6, 12
    ld = (q + k + v + 7) // 8 * 8
    proj, slots = draw(rng, (n, ld), dtype), rng.permutation(rows)[:n].astype(np.int32)
    slots[2] = -1
    kc, vc = torch.full((rows, k), 7.0, device=cuda, dtype=dtype), torch.full((rows, v), 7.0, device=cuda, dtype=dtype)
    got = ops.attn_store(dev_t(proj, cuda), q, k, v, kc, vc, dev_i(slots, cuda), dtype)
    kr, vr = np.full((rows, k), 7.0), np.full((rows, v), 7.0)
    for t in range(n):
        if slots[t] >= 0:
            kr[slots[t]], vr[slots[t]] = proj[t, q:q + k], proj[t, q + k:q + k + v]
    for a, b in ((got, proj[:, :q]), (kc, kr), (vc, vr)):
        np.testing.assert_array_equal(npf(a), b)


# ---- attention with a temperature, a cap and a slope per head --------------------------------------------------------------

def sloped(q, keys, vals, G, scale, cap, q_temp, pos, gate=None):
    """One token: q [H, D], keys / vals of positions 0..pos as [pos + 1, G, *]."""
    H, out = len(q), []
    dist = pos - np.arange(pos + 1)
    for h in range(H):
        g = h // (H // G)
        s = F.capped_scores(keys[:pos + 1, g] @ q[h] * F.query_temperature(pos, q_temp) * scale, cap, F.head_slope(h, H), dist)
        out.append(F.softmax(s) @ vals[:pos + 1, g])
    o = np.concatenate(out)
    return o if gate is None else o * F.sigmoid(gate)


def slopes_of(H):
    return np.array([F.head_slope(h, H) for h in range(H)])


def run_sloped(cuda, rng, dtype, G, bs, scale, cap, q_temp, steps, q, keys, vals, gate=None):
    """One launch holding, per entry of `steps` (prefix length, new tokens), a portion of a sequence of its own; pages in random
    order.  q [tokens, H, D]; keys / vals: one array per sequence."""
    from nano_vllm_rs_b200 import ops
    H, D, V = q.shape[1], q.shape[2], vals[0].shape[2]
    ctxs = [p + n for p, n in steps]
    tables, slot, rows = paged(rng, ctxs, bs)
    kc = torch.zeros((rows, G * D), device=cuda, dtype=dtype); vc = torch.zeros((rows, G * V), device=cuda, dtype=dtype)
    for s, c in enumerate(ctxs):
        idx = torch.tensor([slot(s, j) for j in range(c)], device=cuda)
        kc[idx] = dev_t(keys[s].reshape(c, -1), cuda, dtype); vc[idx] = dev_t(vals[s].reshape(c, -1), cuda, dtype)
    tok_seq = np.concatenate([[s] * n for s, (_, n) in enumerate(steps)]).astype(np.int32)
    pos = np.concatenate([np.arange(p, p + n) for p, n in steps]).astype(np.int64)
    cu = np.concatenate([[0], np.cumsum([n for _, n in steps])]).astype(np.int32)
    got = ops.extended_attention(dev_t(q.reshape(len(pos), -1), cuda, dtype), dev_t(gate, cuda) if gate is not None else None, kc, vc, dev_i(tok_seq, cuda),
                                 dev_i(pos, cuda, torch.int64), dev_i(tables, cuda), bs, H, G, D, V, scale, softcap=cap or 0.0,
                                 temp_coef=q_temp["coef"] if q_temp else 0.0, temp_every=q_temp["every"] if q_temp else 1,
                                 slopes=dev_t(slopes_of(H), cuda), cu_tokens=dev_i(cu, cuda))
    ref = np.stack([sloped(q[t], keys[tok_seq[t]], vals[tok_seq[t]], G, scale, cap, q_temp, int(pos[t]), None if gate is None else gate[t])
                    for t in range(len(pos))])
    return npf(got), ref


SLOPED = [  # heads, kv heads, dim, vdim, page, cap, q_temp
    (4, 2, 6, 5, 16, 3.0, (0.5, 7)), (12, 2, 80, 64, 32, 20.0, (0.3, 64)), (6, 2, 64, 48, 16, 2.0, (0.4, 100)), (2, 2, 128, 128, 32, None, (0.2, 1)),
    (3, 1, 16, 8, 16, 5.0, None), (6, 3, 32, 32, 16, None, None), (16, 2, 64, 64, 64, 50.0, (0.1, 33)), (20, 1, 48, 32, 32, 1.0, (1.0, 16)),
    (1, 1, 1, 1, 16, 4.0, (0.7, 3)), (8, 8, 72, 40, 16, 8.0, (0.3, 50)), (2, 1, 150, 24, 16, 6.0, (0.2, 9)),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", SLOPED)
def test_capped_attention_with_slopes(cuda, dtype, case):
    H, G, D, V, bs, cap, qt = case
    rng = np.random.default_rng(H * 7 + D)
    steps = ((0, 150), (37, 90), (149, 1), (64, 1), (63, 1), (300, 2), (201, 40), (0, 1), (511, 3))
    q_temp = dict(zip(("coef", "every"), qt)) if qt else None
    n = sum(c for _, c in steps)
    q = draw(rng, (n, H, D), dtype)
    keys, vals = [draw(rng, (p + c, G, D), dtype) for p, c in steps], [draw(rng, (p + c, G, V), dtype) for p, c in steps]
    got, ref = run_sloped(cuda, rng, dtype, G, bs, 3.0 / np.sqrt(D), cap, q_temp, steps, q, keys, vals, f32r(rng.standard_normal((n, H * V))))
    tol = 2e-5 if dtype == F32 else 2e-2
    assert np.abs(got - ref).max() < tol * max(1.0, np.abs(ref).max()), np.abs(got - ref).max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [1, 2, 40])
@pytest.mark.parametrize("back,cap,H,bs", [(700, 30.0, 4, 64), (200, 30.0, 8, 16), (65, 25.0, 2, 16), (64, 25.0, 2, 16), (63, 25.0, 2, 64), (1, 20.0, 4, 16),
                                           (0, 20.0, 4, 16), (1100, 40.0, 16, 32)])
def test_one_key_stands_out_against_its_distance(cuda, dtype, portion, back, cap, H, bs):
    """One key per sequence is aligned with the last query (its score sits at the cap), all others score far below: it takes the
    mass of the heads whose slope lets it, and the other heads read near keys.  The slope acts after the cap and on top of the
    distance of every key, pages and tiles apart."""
    rng = np.random.default_rng(back + portion)
    G, D, V, ctx = 1, 64, 16, max(back + 1, portion) + 130
    scale, keys, vals = 0.25, draw(rng, (ctx, G, D), dtype, 0.02), draw(rng, (ctx, G, V), dtype)
    q = draw(rng, (portion, H, D), dtype)
    q[-1] = q[-1, 0]
    keys[ctx - 1 - back, 0] = snap(q[-1, 0] * (3 * cap / (q[-1, 0] @ q[-1, 0] * scale)), dtype)
    got, ref = run_sloped(cuda, rng, dtype, G, bs, scale, cap, None, [(ctx - portion, portion)], q, [keys], [vals])
    tol = 2e-5 if dtype == F32 else 2e-2
    assert np.abs(got - ref).max() < tol * max(1.0, np.abs(ref).max())
    last, hot = got[-1].reshape(H, V), vals[ctx - 1 - back, 0]
    sure = [h for h in range(H) if cap * 0.99 - F.head_slope(h, H) * back > np.log(ctx) + 8]
    for h in sure:
        assert np.abs(last[h] - hot).max() < (1e-3 if dtype == F32 else 3e-2), h
    never = [h for h in range(H) if cap - F.head_slope(h, H) * back < -12]
    for h in never:
        assert np.abs(last[h] - hot).max() > 0.1, h
    assert sure and (back < 500 or never)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [1, 33])
def test_the_cap_comes_before_the_slope(cuda, dtype, portion):
    """Every raw score is far above the cap; only the distances differ, so the weights are those of the slopes alone."""
    rng = np.random.default_rng(portion)
    H, G, D, V, ctx, cap = 4, 2, 16, 8, 300, 2.0
    keys, vals = np.full((ctx, G, D), 4.0), draw(rng, (ctx, G, V), dtype)
    q = np.full((portion, H, D), 4.0)
    got, ref = run_sloped(cuda, rng, dtype, G, 16, 1.0, cap, None, [(ctx - portion, portion)], q, [keys], [vals])
    assert np.abs(got - ref).max() < (2e-5 if dtype == F32 else 2e-2)
    for h in range(H):
        w = np.exp(-F.head_slope(h, H) * (ctx - 1 - np.arange(ctx)))
        np.testing.assert_allclose(got[-1].reshape(H, V)[h], (w / w.sum()) @ vals[:, h // 2], atol=2e-5 if dtype == F32 else 2e-2)


def test_query_temperature_steps(cuda):
    """The temperature of positions around the multiples of `every`, one token per launch, in f32."""
    rng = np.random.default_rng(1)
    H, G, D, V, every = 2, 1, 8, 4, 10
    keys, vals = f32r(rng.standard_normal((45, G, D))), f32r(rng.standard_normal((45, G, V)))
    for p in (0, 8, 9, 10, 18, 19, 20, 28, 29, 44):
        q = f32r(rng.standard_normal((1, H, D)))
        got, ref = run_sloped(cuda, rng, F32, G, 16, 0.5, 5.0, {"coef": 0.8, "every": every}, [(p, 1)], q, [keys[:p + 1]], [vals[:p + 1]])
        np.testing.assert_allclose(got, ref, atol=1e-5, err_msg=str(p))
    assert F.query_temperature(8, {"coef": 0.8, "every": 10}) == 1.0 < F.query_temperature(9, {"coef": 0.8, "every": 10})


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_of_a_sequence_with_slopes(cuda, dtype):
    rng = np.random.default_rng(2)
    H, G, D, V, n = 4, 2, 8, 8, 30
    keys, vals, q = draw(rng, (n, G, D), dtype), draw(rng, (n, G, V), dtype), draw(rng, (n, H, D), dtype)
    for p in range(n):
        got, ref = run_sloped(cuda, rng, dtype, G, 16, 0.6, 3.0, {"coef": 0.4, "every": 4}, [(p, 1)], q[p:p + 1], [keys[:p + 1]], [vals[:p + 1]])
        assert np.abs(got - ref).max() < (1e-5 if dtype == F32 else 2e-2), p


# ---- latent attention ------------------------------------------------------------------------------------------------------

def windowed(q, k, v, pos, size, scale):
    """One token, one head: k, v of positions 0..pos."""
    lo = F.window_start(pos, {"size": size} if size else None)
    return F.softmax(k[lo:pos + 1] @ q * scale) @ v[lo:pos + 1]


TWO_PART = [  # heads, own, shared, vdim, window
    (3, 6, 4, 5, 9), (6, 64, 32, 64, 50), (2, 128, 64, 128, 70), (2, 96, 32, 64, 33), (5, 24, 8, 16, 64), (1, 120, 72, 104, 100), (2, 32, 16, 24, 1), (4, 64, 64, 64, 0),
    (1, 2, 1, 1, 3),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", TWO_PART)
@pytest.mark.parametrize("dense", [True, False])
def test_windowed_attention_with_a_shared_key_part(cuda, dtype, case, dense):
    """Keys [own | shared by the heads], as dense rows of whole prompts and through pages with prefixes."""
    from nano_vllm_rs_b200 import ops
    H, D, sh, V, size = case
    rng = np.random.default_rng(H + D + size)
    steps = [(0, 150), (0, 33), (0, 1), (0, 90)] if dense else [(0, 150), (37, 90), (149, 1), (63, 1), (201, 40)]
    ctxs, scale, bs = [p + n for p, n in steps], 1.5 / np.sqrt(D + sh), 16
    keys, shared, vals = [draw(rng, (c, H, D), dtype) for c in ctxs], [draw(rng, (c, sh), dtype) for c in ctxs], [draw(rng, (c, H, V), dtype) for c in ctxs]
    tok_seq = np.concatenate([[s] * n for s, (_, n) in enumerate(steps)]).astype(np.int32)
    pos = np.concatenate([np.arange(p, p + n) for p, n in steps]).astype(np.int64)
    cu = np.concatenate([[0], np.cumsum([n for _, n in steps])]).astype(np.int32)
    q, gate = draw(rng, (len(pos), H, D + sh), dtype), f32r(rng.standard_normal((len(pos), H * V)))
    ld_s = (sh + 7) // 8 * 8 + 8
    if dense:
        kv = dev_t(np.concatenate([np.concatenate([k.reshape(len(k), -1), v.reshape(len(v), -1)], 1) for k, v in zip(keys, vals)]), cuda, dtype)
        kc, vc, tables = kv[:, :H * D], kv[:, H * D:], None
        ks = torch.zeros((len(pos), ld_s), device=cuda, dtype=dtype)
        ks[:, :sh] = dev_t(np.concatenate(shared), cuda, dtype)
    else:
        tables, slot, rows = paged(rng, ctxs, bs)
        kc, vc, ks = (torch.zeros((rows, c), device=cuda, dtype=dtype) for c in (H * D, H * V, ld_s))
        for s, c in enumerate(ctxs):
            idx = torch.tensor([slot(s, j) for j in range(c)], device=cuda)
            kc[idx], vc[idx] = dev_t(keys[s].reshape(c, -1), cuda, dtype), dev_t(vals[s].reshape(c, -1), cuda, dtype)
            ks[idx, :sh] = dev_t(shared[s], cuda, dtype)
        tables = dev_i(tables, cuda)
    got = npf(ops.extended_attention(dev_t(q.reshape(len(pos), -1), cuda, dtype), dev_t(gate, cuda), kc, vc, dev_i(tok_seq, cuda), dev_i(pos, cuda, torch.int64),
                                     tables, bs, H, H, D + sh, V, scale, window=size, k_shared=ks, shared_dim=sh, cu_tokens=dev_i(cu, cuda)))
    ref = np.zeros((len(pos), H, V))
    for t in range(len(pos)):
        s = tok_seq[t]
        for h in range(H):
            ref[t, h] = windowed(q[t, h], np.concatenate([keys[s][:, h], shared[s]], 1), vals[s][:, h], int(pos[t]), size, scale)
    ref = ref.reshape(len(pos), -1) * F.sigmoid(gate)
    assert np.abs(got - ref).max() < (2e-5 if dtype == F32 else 2e-2) * max(1.0, np.abs(ref).max()), np.abs(got - ref).max()


def folded(cuda, rng, dtype, H, R, rd, size, steps, scale, bs=16, hot=None, workspace=None):
    """Attention over cached [latent | rotated part] rows with the folded queries; hot (sequence 0, last token): a key position whose
    score is made to stand out.  Returns (got, ref, latents of sequence 0)."""
    from nano_vllm_rs_b200 import ops
    ctxs, D, row = [p + n for p, n in steps], 8, (R + rd + 7) // 8 * 8
    lat = [draw(rng, (c, R + rd), dtype, 1.0 if hot is None else 0.05) for c in ctxs]
    tok_seq = np.concatenate([[s] * n for s, (_, n) in enumerate(steps)]).astype(np.int32)
    pos = np.concatenate([np.arange(p, p + n) for p, n in steps]).astype(np.int64)
    qa, q = draw(rng, (len(pos), H, R), dtype), draw(rng, (len(pos), H, D + rd), dtype)
    if hot is not None:
        last = steps[0][1] - 1
        qa[last, :], q[last, :] = qa[last, 0], q[last, 0]
        full = np.concatenate([qa[last, 0], q[last, 0, D:]])
        lat[0][hot] = snap(full * (40.0 / (full @ full * scale)), dtype)
    tables, slot, rows = paged(rng, ctxs, bs)
    cache = torch.zeros((rows, row), device=cuda, dtype=dtype)
    for s, c in enumerate(ctxs):
        cache[torch.tensor([slot(s, j) for j in range(c)], device=cuda), :R + rd] = dev_t(lat[s], cuda, dtype)
    got = npf(ops.latent_rotary_attention(dev_t(qa.reshape(len(pos), -1), cuda), dev_t(q.reshape(len(pos), -1), cuda, dtype), dev_i(tok_seq, cuda),
                                          dev_i(pos, cuda, torch.int64), dev_i(tables, cuda), bs, cache, H, D, rd, R, scale, window=size, workspace=workspace))
    ref = np.stack([np.concatenate([windowed(np.concatenate([qa[t, h], q[t, h, D:]]), lat[tok_seq[t]], lat[tok_seq[t]][:, :R], int(pos[t]), size, scale)
                                    for h in range(H)]) for t in range(len(pos))])
    return got, ref, lat[0][:, :R]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,R,rd,size", [(3, 7, 4, 9), (6, 64, 32, 45), (16, 128, 64, 100), (5, 24, 8, 1), (2, 512, 64, 33), (20, 40, 16, 0), (1, 1, 2, 5)])
def test_folded_latent_attention_with_a_rotated_part(cuda, dtype, H, R, rd, size):
    got, ref, _ = folded(cuda, np.random.default_rng(H + R), dtype, H, R, rd, size, [(0, 100), (37, 50), (149, 1), (64, 1), (300, 2)], 1.5 / np.sqrt(R + rd))
    assert np.abs(got - ref).max() < (2e-5 if dtype == F32 else 2e-2) * max(1.0, np.abs(ref).max()), np.abs(got - ref).max()


def test_long_windows_share_their_keys_over_ctas(cuda):
    """Single tokens in a window of more than a thousand keys: with a workspace their key tiles are split over several CTAs."""
    for H, R, rd, size in ((6, 64, 32, 1200), (3, 128, 8, 2100)):
        ws = torch.zeros(4 * 4 * H * (R + 2), device=cuda)
        got, ref, _ = folded(cuda, np.random.default_rng(R), BF16, H, R, rd, size, [(1500, 1), (2300, 1), (90, 1), (0, 1)], 1.5 / np.sqrt(R + rd), workspace=ws)
        assert np.abs(got - ref).max() < 2e-2 * max(1.0, np.abs(ref).max()), np.abs(got - ref).max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [1, 2, 40, 300])
@pytest.mark.parametrize("size,bs,p", [(41, 64, 420), (64, 16, 383), (63, 16, 384), (33, 32, 351), (1, 16, 340), (128, 16, 511), (5, 16, 303)])
def test_latent_window_edges_stand_out(cuda, dtype, portion, size, bs, p):
    """The last key of the window and the query's own take all the mass when they are made to; the key just outside gets none."""
    tol = 1e-4 if dtype == F32 else 3e-2
    for hot, seen in ((p - size + 1, True), (p, True), (p - size, False)):
        got, ref, lat = folded(cuda, np.random.default_rng(p + size), dtype, 2, 24, 8, size, [(p + 1 - portion, portion)], 0.25, bs, hot)
        last = got[portion - 1].reshape(2, -1)
        assert np.abs(got - ref).max() < tol * max(1.0, np.abs(ref).max()), hot
        assert (np.abs(last - lat[hot]).max() < tol * np.abs(lat[hot]).max()) == seen, hot


# ---- gates, feed-forwards, experts, token inputs -------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,H,V,R", [(5, 3, 5, 7), (64, 4, 32, 128), (70, 2, 64, 64), (1, 1, 1, 1), (33, 16, 128, 512), (3, 2, 8, 24)])
def test_gated_value_projection(cuda, dtype, n, H, V, R):
    from nano_vllm_rs_b200 import ops
    rng = np.random.default_rng(n)
    x, w, gate = draw(rng, (n, H, R), dtype), draw(rng, (H, V, R), dtype, R ** -0.5), f32r(rng.standard_normal((n, H * V + 3)) * 3)
    gd = dev_t(gate, cuda)[:, 2:2 + H * V]
    got = npf(ops.linear_gated(dev_t(x.reshape(n, -1), cuda, dtype), dev_t(w.reshape(H * V, R), cuda, dtype), gd, H, V, R, R, V * R, V))
    pre = np.einsum("nhr,hvr->nhv", x, w).reshape(n, -1)
    tol = dict(rtol=2e-5, atol=2e-5) if dtype == F32 else dict(rtol=1e-2, atol=1e-2)
    np.testing.assert_allclose(got, pre * F.sigmoid(gate[:, 2:2 + H * V]), **tol)
    y = dev_t(pre, cuda, dtype)
    ref = npf(y) * F.sigmoid(gate[:, 2:2 + H * V])
    ops.sigmoid_gate(y, gd)
    np.testing.assert_allclose(npf(y), ref, **tol)
    y8 = dev_t(pre, cuda, dtype)
    ops.sigmoid_gate(y8, gd.contiguous())
    np.testing.assert_array_equal(npf(y8), npf(y))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,layers,layer", [(5, 4, 2), (16, 4, 0), (64, 3, 2), (1, 1, 0), (24, 2, 1), (12, 3, 1)])
def test_token_row_gated_by_the_stream(cuda, dtype, dim, layers, layer):
    from nano_vllm_rs_b200 import ops
    rng = np.random.default_rng(dim)
    n, vocab = 37, 50
    tab, ids = draw(rng, (vocab, dim * layers), dtype), rng.integers(0, vocab, n)
    pad = (dim + 7) // 8 * 8
    gate = f32r(rng.standard_normal((n, pad)) * 4)
    gate[0, 0], gate[1, 0] = 60.0, -60.0
    got = npf(ops.token_gate(dev_t(gate, cuda)[:, :dim], dev_t(tab, cuda, dtype), layer * dim, dev_i(ids, cuda, torch.int64)))
    ref = F.gelu_tanh(gate[:, :dim]) * tab[ids, layer * dim:(layer + 1) * dim]
    np.testing.assert_allclose(got, ref, **(dict(rtol=2e-5, atol=2e-5) if dtype == F32 else dict(rtol=1e-2, atol=1e-2)))


@pytest.mark.parametrize("m", [1, 40, 130, 700])
@pytest.mark.parametrize("inter,k", [(128, 64), (384, 256), (640, 1024), (1024, 2048)])
def test_gelu_gate_in_the_gemm_epilogue(cuda, m, inter, k):
    """Single-CTA, CTA-pair and split-K tiles; both tails of the gate."""
    from nano_vllm_rs_b200 import ops
    rng = np.random.default_rng(m + inter)
    x, w = F.bf16_round(rng.standard_normal((m, k))), F.bf16_round(rng.standard_normal((2 * inter, k)) * 2 / np.sqrt(k))
    w[0], w[1] = F.bf16_round(x[0] * 100.0 / (x[0] @ x[0])), F.bf16_round(-x[0] * 100.0 / (x[0] @ x[0]))
    got = npf(ops.gemm_gated(dev_t(x, cuda, BF16), dev_t(w, cuda, BF16), "gelu"))
    pre = x @ w.T
    np.testing.assert_allclose(got, F.gelu_tanh(pre[:, :inter]) * pre[:, inter:], rtol=2e-2, atol=3e-2)
    assert abs(got[0, 1]) < 1e-20 and abs(got[0, 0] / pre[0, inter] - 100.0) < 2.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,ff", [(7, 24), (3, 5), (33, 256)])
def test_gelu_gate_as_a_kernel(cuda, dtype, n, ff):
    from nano_vllm_rs_b200 import ops
    rng = np.random.default_rng(ff)
    x = draw(rng, (n, 2 * ff), dtype, 3.0)
    x[0, 0], x[0, 1] = 200.0, -200.0
    got = npf(ops.gated_gelu(dev_t(x, cuda, dtype)))
    np.testing.assert_allclose(got, F.gelu_tanh(x[:, :ff]) * x[:, ff:], **(dict(rtol=2e-5, atol=2e-5) if dtype == F32 else dict(rtol=1e-2, atol=1e-2)))


@pytest.mark.parametrize("m", [1, 64, 130, 500])
@pytest.mark.parametrize("n,k", [(32, 4096), (96, 2048), (160, 1024), (256, 4096), (512, 512), (1088, 1024)])
@pytest.mark.parametrize("out", DTYPES)
def test_decode_sized_products_split_the_reduction(cuda, m, n, k, out):
    """Packed projections, gates and routers of few tokens (f32 rows or the operand type): clusters share the reduction."""
    from nano_vllm_rs_b200 import ops
    rng = np.random.default_rng(m + n)
    x, w = F.bf16_round(rng.standard_normal((m, k))), F.bf16_round(rng.standard_normal((n, k)) / np.sqrt(k))
    got = npf(ops.linear(dev_t(x, cuda, BF16), dev_t(w, cuda, BF16), out_dtype=out))
    np.testing.assert_allclose(got, x @ w.T, **(dict(rtol=2e-4, atol=2e-5) if out == F32 else dict(rtol=1e-2, atol=1e-2)))


@pytest.mark.parametrize("E,top", [(5, 2), (16, 1), (3, 3), (1, 1), (100, 7)])
def test_sigmoid_routing(cuda, E, top):
    from nano_vllm_rs_b200 import ops
    rng = np.random.default_rng(E)
    z = f32r(rng.standard_normal((45, E)) * 3)
    z[3] = 1.0                                    # ties: the lowest indices
    idx, w = ops.moe_route_sigmoid(dev_t(z, cuda), None, top)
    for t in range(len(z)):
        o, s = F.route(z[t], top)
        assert idx[t].tolist() == o
        np.testing.assert_allclose(npf(w)[t], s, rtol=1e-6)


@pytest.mark.parametrize("dtype,n,W,ff,E,top", [(F32, 21, 24, 10, 5, 2), (BF16, 21, 24, 10, 5, 2), (BF16, 90, 128, 192, 5, 2), (BF16, 300, 320, 256, 7, 3), (BF16, 40, 64, 64, 3, 1)])
def test_experts_scale_their_input(cuda, dtype, n, W, ff, E, top):
    """The score multiplies what the expert reads (through a nonlinear gate that is not the same as scaling its output)."""
    from nano_vllm_rs_b200 import ops
    rng = np.random.default_rng(n)
    x, gu, dn = draw(rng, (n, W), dtype), draw(rng, (E, 2 * ff, W), dtype, 2.0 / np.sqrt(W)), draw(rng, (E, W, ff), dtype, 1.0 / np.sqrt(ff))
    z = f32r(rng.standard_normal((n, E)) * 2)
    idx, wts = ops.moe_route_sigmoid(dev_t(z, cuda), None, top)
    tensor_cores = W % 64 == 0 and ff % 64 == 0
    row_token, row_w, tile_expert, slot_row = ops.moe_sort_weighted(idx, wts, E, tile_rows=128 if tensor_cores else 32)
    rows, xd = row_token.shape[0], dev_t(x, cuda, dtype)
    gud, dnd = dev_t(gu.reshape(E * 2 * ff, W), cuda, dtype), dev_t(dn.reshape(E * W, ff), cuda, dtype)
    if tensor_cores:
        act = ops.gemm_gated_grouped(xd[row_token.long().clamp(min=0)].contiguous(), gud, tile_expert, ff, E, "silu", row_scale=row_w)
        eo = ops.gemm_bf16_grouped(act, dnd, tile_expert, W, E)
    else:
        act = ops.linear_grouped_scaled(xd, gud, row_token, row_w, tile_expert, rows, ff, W, 2 * ff * W, glu=3)
        eo = ops.linear_grouped(act, dnd, None, tile_expert, rows, W, ff, W * ff)
    got = npf(ops.moe_combine(eo, xd, None, idx, None, slot_row, E))
    ref, wrong = np.zeros((n, W)), np.zeros((n, W))
    for t in range(n):
        for e, s in zip(*F.route(z[t], top)):
            f = lambda y: dn[e] @ (F.silu(gu[e, :ff] @ y) * (gu[e, ff:] @ y))
            ref[t] += f(s * x[t]); wrong[t] += s * f(x[t])
    tol = 1e-4 if dtype == F32 else 3e-2
    np.testing.assert_allclose(got, ref, rtol=tol, atol=tol * max(1.0, np.abs(ref).max()))
    assert np.abs(wrong - ref).max() > 3 * tol * max(1.0, np.abs(ref).max())


# ------------------------------------------------------------------------------------------------ the engine

TOL = 2e-4


def within(errs, dtype, routed=True):
    """errs: row errors of one or more requests.  f32: every position to rounding.  bf16 without routers: operand rounding only.
    bf16 with routers: a close call of a router (and, in the narrowest models, a sublayer's output that is nearly zero before its
    norm) moves single rows and, less, those that later read them; a fault would move most of them."""
    e = np.concatenate(errs)
    if not np.isfinite(e).all():
        return False
    if dtype == "float32":
        return e.max() < TOL
    if not routed:
        return e.max() < 0.12 and e.mean() < 0.03
    return np.median(e) < 0.08 and (e > 0.3).mean() < 0.1


def variant(name):
    A, L, dense, moe = F.attention_mixer, F.latent_mixer, F.dense_mlp, F.expert_mlp
    if name == "all_kinds":      # every mixer with every feed-forward, sizes all different
        return F.make_config([("latent_attention", L(), moe()), ("attention", A(), dense(20)),
                              ("attention", A(heads=6, kv_heads=3, dim=10, vdim=12, softcap=8.0, coef=0.2, every=11, scale=0.3), moe(ff=6, experts=3, top=3)),
                              ("latent_attention", L(heads=2, dim=12, rot_dim=6, vdim=9, q_rank=5, kv_rank=14, size=20, base=1e4, scaling=(5.0, 16.0, 2.0, 300)), None),
                              ("attention", A(heads=3, kv_heads=1, dim=5, vdim=4, softcap=1.5, coef=1.0, every=1), None),
                              ("latent_attention", L(heads=5, dim=3, rot_dim=2, vdim=2, size=3, scaling=None), dense(12))])
    if name == "ones":           # sizes that are 1 or equal to one another, a window of one and one of everything, parts left out
        return F.make_config([("attention", A(heads=1, kv_heads=1, dim=1, vdim=1, softcap=1.0, coef=1.0, every=1, scale=1.0), moe(ff=1, experts=1, top=1)),
                              ("latent_attention", L(heads=1, dim=1, rot_dim=2, vdim=1, q_rank=1, kv_rank=1, size=1, scale=1.0, base=2.0, scaling=(1.0, 1.0, 1.0, 1)), dense(1)),
                              ("latent_attention", L(heads=8, dim=8, rot_dim=8, vdim=8, q_rank=8, kv_rank=8, size=1000, scaling=(8.0, 8.0, 8.0, 8)), moe(ff=8, experts=8, top=8)),
                              ("attention", A(heads=8, kv_heads=8, dim=8, vdim=8, softcap=None, coef=None), dense(8)),
                              ("latent_attention", L(size=None), None)], width=16, vocab=33, side_dim=1)
    if name == "tensor_core":    # sizes the tensor-core kernels accept (bf16): width and inner sizes multiples of 64, heads of 64 to 192
        return F.make_config([("attention", A(heads=6, kv_heads=3, dim=64, vdim=64, softcap=20.0, coef=0.3, every=20, scale=0.2), dense(256)),
                              ("latent_attention", L(heads=5, dim=64, rot_dim=32, vdim=64, q_rank=64, kv_rank=128, size=30, scale=0.12, base=1e4, scaling=(4.0, 8.0, 1.0, 90)), moe(ff=64, experts=4, top=2)),
                              ("attention", A(heads=8, kv_heads=1, dim=128, vdim=80, softcap=4.0, coef=0.1, every=7, scale=0.15), moe(ff=128, experts=3, top=1)),
                              ("latent_attention", L(heads=2, dim=128, rot_dim=64, vdim=128, q_rank=128, kv_rank=64, size=70, scale=0.08, scaling=(2.0, 4.0, 1.0, 500)), dense(128))],
                             width=128, vocab=96, side_dim=64)
    if name == "mid":            # sizes between: a width that is no power of two, heads of 48 and 24
        return F.make_config([("latent_attention", L(heads=6, dim=48, rot_dim=24, vdim=40, q_rank=72, kv_rank=56, size=25, scale=0.14, scaling=(6.0, 5.0, 1.5, 40)), dense(192)),
                              ("attention", A(heads=9, kv_heads=3, dim=48, vdim=24, softcap=6.0, coef=0.5, every=13, scale=0.2), moe(ff=96, experts=6, top=3)),
                              ("attention", A(heads=4, kv_heads=4, dim=24, vdim=56, softcap=12.0, coef=0.2, every=30, scale=0.25), dense(100)),
                              ("latent_attention", L(heads=3, dim=40, rot_dim=16, vdim=72, q_rank=24, kv_rank=88, size=64, scale=0.13), moe(ff=64, experts=3, top=2))],
                             width=192, vocab=200, side_dim=24)
    if name == "no_router":      # odd sizes of a less narrow model, dense feed-forwards only: every position is comparable in bf16 too
        return F.make_config([("latent_attention", L(heads=3, dim=18, rot_dim=10, vdim=14, q_rank=30, kv_rank=26, size=9, scale=0.2), dense(90)),
                              ("attention", A(heads=4, kv_heads=2, dim=22, vdim=18, softcap=8.0, coef=0.2, every=11, scale=0.2), dense(70)),
                              ("latent_attention", L(heads=5, dim=12, rot_dim=6, vdim=13, q_rank=25, kv_rank=34, size=20, scale=0.25, scaling=(5.0, 16.0, 2.0, 300)), None),
                              ("attention", A(heads=6, kv_heads=3, dim=15, vdim=11, softcap=4.0, coef=0.5, every=3, scale=0.25), dense(50))],
                             width=60, vocab=90, side_dim=21)
    raise KeyError(name)


VARIANTS = ["all_kinds", "ones", "tensor_core", "mid", "no_router"]


def model_for(name, rng):
    cfg = variant(name)
    return cfg, F.random_weights(cfg, rng)


def make_engine(tmp_path, cfg, w, dtype, **kw):
    d = write_checkpoint(tmp_path / ("m_" + dtype), cfg, w, F.to_bf16_bits)
    return engine_on(d, dtype, **kw), d


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", VARIANTS)
def test_engine_schedules_match_the_oracle(cuda, tmp_path, name, dtype):
    rng = np.random.default_rng(500 + VARIANTS.index(name))
    cfg, w = model_for(name, rng)
    lens = [1, 2, 37, 90, 33]
    reqs = [rng.integers(0, cfg["vocab"], n).tolist() for n in lens]
    ref = [F.run_sequence(cfg, w, r) for r in reqs]
    eng, _ = make_engine(tmp_path, cfg, w, dtype, bs=16, blocks=12)    # 192 slots: the requests only fit one after another
    routed = name != "no_router"

    def check(got, want, what):
        errs = [rel_err(got[i], np.asarray(want[i], np.float64)) for i in got]
        assert within(errs, dtype, routed), f"{name} {dtype} {what}: per request, largest {[float(e.max()) for e in errs]}, median {[float(np.median(e)) for e in errs]}"

    whole = replay(eng, reqs, [[(i, len(r))] for i, r in enumerate(reqs)])
    check(whole, ref, "whole prompts")
    # most of the prompt at once, the last tokens one by one (windows and page borders pass under decoded tokens)
    dec = replay(eng, reqs, [s for i, r in enumerate(reqs) for s in ([[(i, max(1, len(r) - 50))]] + [[(i, 1)]] * (len(r) - max(1, len(r) - 50)))])
    check(dec, ref, "prefill + single tokens")
    check(replay(eng, reqs[:3], [[(i, 1)] for i, r in enumerate(reqs[:3]) for _ in r]), ref, "single tokens only")
    por = replay(eng, reqs, [[(i, c)] for i, r in enumerate(reqs) for c in cut(len(r), [2, 5, 16, 3, 17, 2, 31])])
    check(por, ref, "portions")
    check(replay(eng, reqs, [[(i, c)] for i, r in enumerate(reqs) for c in cut(len(r), [2])]), ref, "portions of two")
    # a position must not depend on how the prompt was cut, beyond rounding
    check(por, whole, "portions against whole prompts"); check(dec, whole, "single tokens against whole prompts")


@pytest.mark.parametrize("name", ["all_kinds", "mid"])
def test_engine_layer_taps_match_the_oracle(cuda, tmp_path, name):
    """The residual stream after every layer, for a prompt: each mixer and feed-forward kind is checked where it sits."""
    from nano_vllm_rs_b200.engine import SamplingParams
    rng = np.random.default_rng(51)
    cfg, w = model_for(name, rng)
    toks = rng.integers(0, cfg["vocab"], 30).tolist()
    _, taps = F.run_sequence(cfg, w, toks, layer_taps=True)
    eng, _ = make_engine(tmp_path, cfg, w, "float32")
    tap = eng.model_runner.layer_tap(len(toks))
    sid = eng.scheduler.add_sequence(toks, SamplingParams(temperature=0.0, max_tokens=1, ignore_eos=True))
    eng.step_chunks([sid], [len(toks)], [0])
    for i in range(len(cfg["layers"])):
        np.testing.assert_allclose(tap[i], taps[i], rtol=2e-4, atol=2e-4, err_msg="after layer %d" % i)


@pytest.mark.parametrize("name,dtype", [("all_kinds", "float32"), ("all_kinds", "bfloat16"), ("no_router", "bfloat16")])
def test_engine_mixed_batches_reuse_pages(cuda, tmp_path, name, dtype):
    """Up to four live requests per step, portions of some beside single tokens of others, in a pool that only holds them
    because finished requests give their pages back; every request equals its run alone and the oracle."""
    rng = np.random.default_rng(52)
    cfg, w = model_for(name, rng)
    lens = [50, 23, 64, 9, 41, 30, 17]
    reqs = [rng.integers(0, cfg["vocab"], n).tolist() for n in lens]
    ref = [F.run_sequence(cfg, w, r) for r in reqs]
    eng, _ = make_engine(tmp_path, cfg, w, dtype, bs=16, blocks=11, max_seqs=4)   # 176 slots < 234 tokens in total
    need = [(n + 15) // 16 for n in lens]
    at, live, nxt, sched, k = [0] * len(lens), [], 0, [], 0
    while nxt < len(reqs) or live:
        while nxt < len(reqs) and len(live) < 4 and sum(need[i] for i in live) + need[nxt] <= 11:
            live.append(nxt); nxt += 1
        step = []
        for i in live:
            k += 1
            if k % 5 == 0 and len(live) > 1:
                continue                                  # a live request may sit a step out
            c = 1 if (at[i] > lens[i] // 2 or k % 3 == 0) else [2, 7, 16, 5][k % 4]
            c = min(c, lens[i] - at[i])
            step.append((i, c)); at[i] += c
        if step:
            sched.append(step)
        live = [i for i in live if at[i] < lens[i]]
    assert any(len(s) == 4 for s in sched) and any(len({c for _, c in s}) > 1 for s in sched)
    mixed = replay(eng, reqs, sched)
    st = eng.scheduler.get_stats()
    assert st["free_blocks"] == st["total_blocks"] == 11
    alone = replay(eng, reqs, [[(i, len(r))] for i, r in enumerate(reqs)])
    for want in (ref, alone):
        errs = [rel_err(mixed[i], np.asarray(want[i], np.float64)) for i in range(len(reqs))]
        assert within(errs, dtype, name != "no_router"), [float(e.max()) for e in errs]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_engine_long_decoding(cuda, tmp_path, dtype):
    """300 tokens at once, then 80 one by one over 20+ pages: windows of 70 and 33 pass over decoded tokens while attention layers
    reach hundreds of tokens back, and the query temperature steps on."""
    rng = np.random.default_rng(53)
    A, L = F.attention_mixer, F.latent_mixer
    cfg = F.make_config([("attention", A(heads=4, softcap=6.0, every=64), F.dense_mlp(16)), ("latent_attention", L(size=70), None),
                         ("latent_attention", L(size=33, heads=2, scaling=(2.0, 8.0, 1.0, 200)), F.dense_mlp(16)), ("attention", A(softcap=None, every=100), F.expert_mlp())])
    w = F.random_weights(cfg, rng)
    toks = rng.integers(0, cfg["vocab"], 380).tolist()
    eng, _ = make_engine(tmp_path, cfg, w, dtype, bs=16, blocks=24, max_seqs=2)
    e = rel_err(replay(eng, [toks], [[(0, 300)]] + [[(0, 1)]] * 80)[0], F.run_sequence(cfg, w, toks))
    assert within([e], dtype), (int(e.argmax()), e.max(), np.median(e))


def test_engine_whole_prompts_and_portions_agree_in_bf16(cuda, tmp_path):
    """Long prompts take the form with keys and values per head, portions and single tokens the folded one, large portions one GEMM
    per head: the same logits, within bf16 rounding, on heads of 64 + 32 and 128 + 64 values."""
    rng = np.random.default_rng(54)
    cfg = variant("tensor_core")
    cfg["layers"] = [dict(l, mlp=F.dense_mlp(128)) for l in cfg["layers"]]     # no router: every position is comparable
    w = F.random_weights(cfg, rng)
    reqs = [rng.integers(0, cfg["vocab"], n).tolist() for n in (700, 300)]
    eng, _ = make_engine(tmp_path, cfg, w, "bfloat16", bs=64, blocks=20)
    whole = replay(eng, reqs, [[(0, 700), (1, 300)]])
    for sched in ([[(0, 650), (1, 40)], [(0, 50), (1, 260)]], [[(0, 20)], [(0, 620), (1, 2)], [(1, 298), (0, 1)]] + [[(0, 1)]] * 59,
                  [[(0, 130)], [(0, 570), (1, 299)], [(1, 1)]]):
        got = replay(eng, reqs, sched)
        for i in range(2):
            e = rel_err(got[i], whole[i].astype(np.float64))
            assert e.max() < 0.1 and e.mean() < 0.03, (i, int(e.argmax()), e.max(), e.mean())
    e = rel_err(whole[1], F.run_sequence(cfg, w, reqs[1]))
    assert e.max() < 0.1 and e.mean() < 0.03, (e.max(), e.mean())


def greedy(cfg, w, prompt, n_new):
    """The oracle's greedy continuation and the top-1 / top-2 margin of every step (relative to the row's spread)."""
    seq, out, margins, lg = F.Sequence(cfg), [], [], None
    for t in prompt:
        lg = F.token_step(cfg, w, seq, int(t))
    for _ in range(n_new):
        o = np.argsort(lg)
        out.append(int(o[-1])); margins.append((lg[o[-1]] - lg[o[-2]]) / lg.std())
        lg = F.token_step(cfg, w, seq, out[-1])
    return out, margins


def agreement(got, ref, margins, floor):
    """Tokens until the first difference, which must be a near-tie."""
    for j, (a, b) in enumerate(zip(got, ref)):
        if a != b:
            assert margins[j] < floor, (j, margins[j])
            return j
    return len(got)


@pytest.mark.parametrize("name,dtype", [("all_kinds", "float32"), ("no_router", "bfloat16")])
def test_greedy_generation_through_the_engine(cuda, tmp_path, name, dtype):
    """LLMEngine.generate: the scheduler's own prefill / decode batches, decode steps replayed as CUDA graphs, pages taken and
    returned, six prompts (two with a common first page) for four sequences at a time."""
    from nano_vllm_rs_b200.engine import SamplingParams
    rng = np.random.default_rng(55)
    cfg, w = model_for(name, rng)
    head = rng.integers(0, cfg["vocab"], 16).tolist()
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (5, 1)] + [head + rng.integers(0, cfg["vocab"], n).tolist() for n in (14, 5)] + \
              [rng.integers(0, cfg["vocab"], n).tolist() for n in (3, 20)]
    n_new = 40
    eng, _ = make_engine(tmp_path, cfg, w, dtype, bs=16, blocks=40, max_seqs=4, eager=0)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=n_new, ignore_eos=True))
    agreed = 0
    for p, o in zip(prompts, outs):
        assert len(o) == n_new
        agreed += agreement(o, *greedy(cfg, w, p, n_new), 1e-3 if dtype == "float32" else 0.2)
    assert agreed > (0.9 if dtype == "float32" else 0.3) * n_new * len(prompts), agreed
    st = eng.scheduler.get_stats()
    assert st["decode_batches"] >= n_new - 1 and st["free_blocks"] == st["total_blocks"]


def test_generation_survives_preemption(cuda, tmp_path):
    """Four prompts with a common first page in a pool too small for them to grow: a victim loses its pages and is recomputed; the
    tokens stay the oracle's."""
    from nano_vllm_rs_b200.engine import SamplingParams
    rng = np.random.default_rng(56)
    cfg, w = model_for("all_kinds", rng)
    head = rng.integers(0, cfg["vocab"], 16).tolist()
    prompts = [head + rng.integers(0, cfg["vocab"], n).tolist() for n in (1, 6, 3, 9)]
    eng, _ = make_engine(tmp_path, cfg, w, "float32", bs=16, blocks=8, max_seqs=4, eager=0)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True))
    st = eng.scheduler.get_stats()
    assert st["preemptions"] > 0 and st["free_blocks"] == st["total_blocks"]
    for p, o in zip(prompts, outs):
        agreement(o, *greedy(cfg, w, p, 40), 1e-3)


def test_model_without_token_inputs(cuda, tmp_path):
    """A configuration without the side table has no tensors of it, and its layers end with the feed-forward."""
    rng = np.random.default_rng(57)
    cfg = F.make_config([("attention", F.attention_mixer(), F.dense_mlp()), ("latent_attention", F.latent_mixer(), None)])
    w = F.random_weights(cfg, rng)
    for i in range(2):
        w["l%d.side.norm" % i] = np.zeros(cfg["width"])           # the oracle's token input adds nothing
    toks = rng.integers(0, cfg["vocab"], 20).tolist()
    ref = F.run_sequence(cfg, w, toks)
    plain = {k: v for k, v in cfg.items() if k != "token_side"}
    eng = engine_on(write_checkpoint(tmp_path / "plain", plain, {k: v for k, v in w.items() if "side" not in k}, F.to_bf16_bits), "float32")
    assert rel_err(replay(eng, [toks], [[(0, 20)]])[0], ref).max() < TOL


def test_synthetic_weights_and_command_line(cuda, tmp_path):
    """Seeded synthetic weights (no checkpoint) run a step; `python -m nano_vllm_rs_b200 generate` on a checkpoint gives the
    oracle's greedy tokens and, with a temperature, draws of the device sampler; the registry lists the architecture."""
    from nano_vllm_rs_b200.engine import Config, LLMEngine, SamplingParams
    rng = np.random.default_rng(58)
    cfg = variant("tensor_core")
    eng = LLMEngine(Config(model_config=cfg, dtype="bfloat16", kvcache_block_size=16, num_kvcache_blocks=8, max_num_seqs=2,
                           max_num_batched_tokens=128, max_model_len=128, enforce_eager=1), init_weights=True)
    sid = eng.scheduler.add_sequence(rng.integers(0, cfg["vocab"], 20).tolist(), SamplingParams(temperature=0.0, max_tokens=1, ignore_eos=True))
    lg = eng.step_chunks([sid], [20], [19])
    assert np.isfinite(lg).all() and lg.std() > 0
    cfg, w = model_for("all_kinds", rng)
    model_dir = write_checkpoint(tmp_path / "cli", cfg, w, F.to_bf16_bits)
    prompt = rng.integers(0, cfg["vocab"], 9).tolist()
    run = lambda *extra: subprocess.run([sys.executable, "-m", "nano_vllm_rs_b200", "generate", "--model", model_dir, "--dtype", "float32", "--prompt-ids",
                                         ",".join(map(str, prompt)), "--max-tokens", "12", "--block-size", "16", *extra], cwd=ROOT, capture_output=True,
                                        text=True, timeout=600)
    r = run()
    assert r.returncode == 0, r.stderr[-2000:]
    ref, margins = greedy(cfg, w, prompt, 12)
    agreement(json.loads(r.stdout.strip().splitlines()[-1])["completion_ids"], ref, margins, 1e-3)
    r = run("--temperature", "1.5", "--top-k", "20")      # the device sampler draws from the same logits
    assert r.returncode == 0, r.stderr[-2000:]
    sampled = json.loads(r.stdout.strip().splitlines()[-1])["completion_ids"]
    assert len(sampled) == 12 and all(0 <= t < cfg["vocab"] for t in sampled)
    r = subprocess.run([sys.executable, "-m", "nano_vllm_rs_b200", "architectures"], cwd=ROOT, capture_output=True, text=True, timeout=120)
    assert "Fomerax" in r.stdout


def test_foreign_and_missing_tensors_are_refused(cuda, tmp_path):
    from nano_vllm_rs_b200 import _ffi
    rng = np.random.default_rng(59)
    cfg = F.make_config([("attention", F.attention_mixer(), None)])
    w = F.random_weights(cfg, rng)
    with pytest.raises(_ffi.NvllmError) as e:
        engine_on(write_checkpoint(tmp_path / "more", cfg, {**w, "l0.mix.sink": np.zeros(4)}, F.to_bf16_bits), "float32")
    assert "l0.mix.sink" in str(e.value)
    with pytest.raises(_ffi.NvllmError) as e:
        engine_on(write_checkpoint(tmp_path / "shape", cfg, {**w, "l0.side.gate": np.zeros((3, cfg["width"]))}, F.to_bf16_bits), "float32")
    assert "l0.side.gate" in str(e.value)


def test_trace_run_replays_a_schedule(cuda, tmp_path):
    rng = np.random.default_rng(60)
    cfg, w = model_for("all_kinds", rng)
    model_dir = write_checkpoint(tmp_path / "trace", cfg, w, F.to_bf16_bits)
    a, b = rng.integers(0, cfg["vocab"], 70).tolist(), rng.integers(0, cfg["vocab"], 9).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:8], "want": []}, {"id": "a", "tokens": a[40:69], "want": [28]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[69:], "want": [0]}, {"id": "b", "tokens": b[8:], "want": [0]}], "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b, "want": [8]}], "end": ["c"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", model_dir, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    ra, rb = F.run_sequence(cfg, w, a), F.run_sequence(cfg, w, b)
    rd = lambda n: np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
    for got, ref in ((rd(0), ra[[0, 39]]), (rd(1), ra[[68]]), (rd(2), np.stack([ra[69], rb[8]])), (rd(3), rb[[8]])):
        assert got.shape == ref.shape and rel_err(got, ref).max() < TOL
