"""CPU tests around the Fomerax integration: properties of the oracle's mechanisms that hold by construction (so that the
yardstick itself is pinned), the model registry's configuration reader, and the scheduler's pages."""
import json
import math

import numpy as np
import pytest

from oracle import fomerax as F


def small_cfg(**kw):
    return F.make_config([("latent_attention", F.latent_mixer(), F.dense_mlp(10)), ("attention", F.attention_mixer(), F.expert_mlp()),
                          ("latent_attention", F.latent_mixer(heads=2, size=4), None), ("attention", F.attention_mixer(heads=6), F.dense_mlp())], **kw)


# ------------------------------------------------------------------------------------------------ oracle properties

def test_gelu_and_softmax():
    z = np.array([-30.0, -1.0, 0.0, 0.5, 30.0])
    ref = [0.5 * t * (1 + math.tanh(math.sqrt(2 / math.pi) * (t + 0.044715 * t ** 3))) for t in z]
    np.testing.assert_allclose(F.gelu_tanh(z), ref)
    np.testing.assert_allclose(F.softmax(np.array([1000.0, 1000.0])), [0.5, 0.5])


def test_yarn_keeps_fast_pairs_and_slows_the_others():
    s = {"factor": 4.0, "fast": 8.0, "slow": 1.0, "original": 512}
    f, amp = F.yarn_frequencies(1e4, 32, s)
    plain, one = F.yarn_frequencies(1e4, 32, None)
    assert one == 1.0 and abs(amp - (0.1 * math.log(4.0) + 1.0)) < 1e-15
    at = lambda t: 32 * math.log(512 / (2 * math.pi * t)) / (2 * math.log(1e4))
    lo, hi = math.floor(at(8.0)), math.ceil(at(1.0))
    assert 0 < lo < hi < 16
    np.testing.assert_allclose(f[:lo + 1], plain[:lo + 1]); np.testing.assert_allclose(f[hi:], plain[hi:] / 4.0)
    mid = lo + 1
    r = (mid - lo) / (hi - lo)
    np.testing.assert_allclose(f[mid], plain[mid] * (1 - r) + plain[mid] / 4.0 * r)
    same, amp1 = F.yarn_frequencies(1e4, 32, dict(s, factor=1.0))
    np.testing.assert_allclose(same, plain); assert amp1 == 1.0
    step, _ = F.yarn_frequencies(50.0, 8, {"factor": 2.0, "fast": 1.0, "slow": 1.0, "original": 100})   # a ramp of width 0 or 1: never a division by zero
    assert np.isfinite(step).all()


def test_rotation_pairs_neighbours_and_depends_on_distance_only():
    rng = np.random.default_rng(1)
    q, k = rng.standard_normal(6), rng.standard_normal(6)
    s = {"factor": 2.0, "fast": 4.0, "slow": 1.0, "original": 40}
    d = lambda pq, pk: F.rotate_pairs(q, pq, 300.0, s) @ F.rotate_pairs(k, pk, 300.0, s)
    assert abs(d(17, 5) - d(112, 100)) < 1e-9 and abs(d(17, 5) - d(17, 6)) > 1e-6
    r = F.rotate_pairs(q, 3, 300.0)
    np.testing.assert_allclose(r[:2], [q[0] * np.cos(3.0) - q[1] * np.sin(3.0), q[1] * np.cos(3.0) + q[0] * np.sin(3.0)])
    amp = 0.1 * math.log(2.0) + 1.0
    np.testing.assert_allclose(F.rotate_pairs(q, 0, 300.0, s), amp * q)


def test_temperature_slope_and_cap():
    t = {"coef": 0.5, "every": 10}
    assert F.query_temperature(8, t) == 1.0 and F.query_temperature(123, None) == 1.0
    assert F.query_temperature(9, t) == 1 + 0.5 * math.log(2) == F.query_temperature(18, t) and F.query_temperature(19, t) == 1 + 0.5 * math.log(3)
    assert F.head_slope(0, 8) == 0.5 and F.head_slope(7, 8) == 2.0 ** -8 and F.head_slope(0, 3) == 2.0 ** (-8 / 3)
    s = F.capped_scores(np.array([1e9, 0.0]), 5.0, 0.25, np.array([40, 2]))
    np.testing.assert_allclose(s, [5.0 - 10.0, -0.5])                       # the slope is taken off after the cap: it is not capped itself
    np.testing.assert_allclose(F.capped_scores(np.array([7.0]), None, 0.5, np.array([2])), [6.0])


def test_windows_and_routing():
    assert [F.window_start(p, {"size": 4}) for p in (0, 3, 4, 20)] == [0, 0, 1, 17]
    assert F.window_start(9, {"size": 1}) == 9 and F.window_start(9, None) == 0 and F.window_start(9, {}) == 0
    o, s = F.route(np.array([0.0, 2.0, 2.0, -1.0]), 3)
    assert o == [1, 2, 0]
    np.testing.assert_allclose(s, [1 / (1 + math.exp(-2)), 1 / (1 + math.exp(-2)), 0.5])    # not renormalised


def test_scores_scale_the_experts_input():
    rng = np.random.default_rng(2)
    cfg = F.make_config([("attention", F.attention_mixer(), F.expert_mlp(experts=1, top=1))])
    w = F.random_weights(cfg, rng)
    x = rng.standard_normal(24)
    s = float(F.sigmoid(w["l0.mlp.router"] @ x)[0])
    f = lambda y: w["l0.mlp.e0.down"] @ (F.silu(w["l0.mlp.e0.gate"] @ y) * (w["l0.mlp.e0.up"] @ y))
    got = F.expert_ff(w, "l0.", cfg["layers"][0]["mlp"], x)
    np.testing.assert_allclose(got, f(s * x))
    assert np.abs(got - s * f(x)).max() > 1e-3


def test_token_input_reads_its_own_layers_part_of_the_row():
    rng = np.random.default_rng(3)
    cfg = F.make_config([("attention", F.attention_mixer(), None), ("attention", F.attention_mixer(), None)])
    w = F.random_weights(cfg, rng)
    _, base = F.run_sequence(cfg, w, [7], layer_taps=True)
    w2 = dict(w); w2["side.embed"] = w["side.embed"].copy()
    w2["side.embed"][7, 5:] *= -2.0                                        # the second layer's part of token 7
    _, other = F.run_sequence(cfg, w2, [7], layer_taps=True)
    np.testing.assert_array_equal(other[0], base[0]); assert np.abs(other[1] - base[1]).max() > 1e-3
    _, unread = F.run_sequence(cfg, w2, [8], layer_taps=True)
    np.testing.assert_array_equal(unread, F.run_sequence(cfg, w, [8], layer_taps=True)[1])


def test_what_a_token_reaches():
    """A latent layer forgets what leaves its window; an attention layer does not."""
    rng = np.random.default_rng(5)
    toks = rng.integers(0, 80, 14).tolist()
    swap = toks[:3] + [(toks[3] + 1) % 80] + toks[4:]
    for kind, mixer, far in (("latent_attention", F.latent_mixer(size=4), False), ("attention", F.attention_mixer(), True)):
        cfg = F.make_config([(kind, mixer, F.dense_mlp(8))])
        w = F.random_weights(cfg, rng)
        moved = np.abs(F.run_sequence(cfg, w, toks) - F.run_sequence(cfg, w, swap)).max(-1)
        assert moved[:3].max() == 0 and moved[3:7].min() > 1e-6 and (moved[7:].min() > 1e-9 if far else moved[7:].max() < 1e-12)
    cfg = F.make_config([("latent_attention", F.latent_mixer(size=4), None)])
    w = F.random_weights(cfg, rng)
    off = dict(cfg, layers=[dict(cfg["layers"][0], mixer=dict(cfg["layers"][0]["mixer"], mask={"size": 5}))])
    d = np.abs(F.run_sequence(cfg, w, toks) - F.run_sequence(off, w, toks)).max(-1)
    assert d[:4].max() == 0 and d[4:].min() > 1e-6                         # one token more in the window shows as soon as it exists


# ------------------------------------------------------------------------------------------------ registry, scheduler

def test_model_registry_reads_config_json():
    from nano_vllm_rs_b200.engine import Config, lib
    assert b"Fomerax" in lib().nvllm_registered_architectures()
    c = Config(model_config=json.dumps(small_cfg(vocab=77, width=24)))
    assert (c.arch, c.vocab_size, c.hidden_size, c.num_hidden_layers, c.recurrent_state) == ("Fomerax", 77, 24, 4, 0)
    plain = small_cfg()
    plain.pop("token_side")
    assert Config(model_config=json.dumps(plain)).arch == "Fomerax"


@pytest.mark.parametrize("breakage,needle", [
    (lambda c: c["layers"][0].update(type="linear"), "linear"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "heads"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=513), "vdim"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), "rot dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6), "rot dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0), "scaling"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=1.0), "base"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"].update(kv_rank=2000), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=-1), "mask size"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "sparse"),
    (lambda c: c["layers"][0]["mlp"].update(ff=0), "feed-forward size"),
    (lambda c: c["token_side"].update(dim=0), "token_side"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
])
def test_bad_model_configs_are_refused_with_a_reason(breakage, needle):
    from nano_vllm_rs_b200 import _ffi
    from nano_vllm_rs_b200.engine import Config
    cfg = small_cfg()
    breakage(cfg)
    with pytest.raises(_ffi.NvllmError) as e:
        Config(model_config=json.dumps(cfg))
    assert needle in str(e.value)


def test_portion_steps_take_pages_and_return_them():
    from nano_vllm_rs_b200.engine import Config, SamplingParams, Scheduler
    cfg = Config(model_config=json.dumps(small_cfg()), kvcache_block_size=16, num_kvcache_blocks=4, max_num_seqs=2,
                 max_num_batched_tokens=64, max_model_len=64)
    s = Scheduler(cfg)
    sp = SamplingParams(temperature=0.0, max_tokens=1, ignore_eos=True)
    a, b = s.add_sequence(list(range(20)), sp), s.add_sequence(list(range(30)), sp)
    s.schedule_chunks([a, b], [17, 2]); s.commit_chunks()
    s.schedule_chunks([a, b], [3, 28]); s.commit_chunks()           # every page is in use
    s.finish_sequence(a); s.release_sequence(a)
    c = s.add_sequence(list(range(32)), sp)
    batch = s.schedule_chunks([c], [32])
    assert len(set((np.asarray(batch.slot_mapping) // 16).tolist())) == 2
