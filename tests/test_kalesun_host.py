"""CPU tests around the Kalesun integration: properties of the oracle's mechanisms that hold by construction (so that the
yardstick itself is pinned), the model registry's configuration reader, and the scheduler's pages and state slots."""
import json
import math

import numpy as np
import pytest

from oracle import kalesun as K


def small_cfg(**kw):
    return K.make_config([("gla", K.gla_mixer(), K.dense_mlp(10)), ("attention", K.attention_mixer(v_mix=True), K.expert_mlp()),
                          ("delta", K.delta_mixer(), None), ("attention", K.attention_mixer(heads=6, v_mix=True), K.dense_mlp())], **kw)


# ------------------------------------------------------------------------------------------------ oracle properties

def test_visible_keys_are_the_window_and_the_kept_first_ones():
    m = {"size": 4, "keep_first": 2}
    assert K.visible_keys(0, m) == [0] and K.visible_keys(3, m) == [0, 1, 2, 3] and K.visible_keys(5, m) == [0, 1, 2, 3, 4, 5]
    assert K.visible_keys(6, m) == [0, 1, 3, 4, 5, 6] and K.visible_keys(20, m) == [0, 1, 17, 18, 19, 20]
    assert K.visible_keys(9, {"size": 1, "keep_first": 0}) == [9] and K.visible_keys(2, {"size": 1, "keep_first": 8}) == [0, 1, 2]
    assert K.visible_keys(5, None) == list(range(6)) and K.visible_keys(5, {"size": 2}) == [4, 5]


def test_frequencies_keep_ramp_or_slow_down_by_wavelength():
    s = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 100}
    wave = lambda l: 2 * math.pi / l
    assert K.scaled_frequency(wave(33.0), s) == wave(33.0)                       # shorter than 100 / 3
    assert K.scaled_frequency(wave(101.0), s) == wave(101.0) / 4.0               # longer than 100
    f = wave(50.0)                                                               # 2 turns: halfway between 1 and 3
    np.testing.assert_allclose(K.scaled_frequency(f, s), 0.5 * f / 4.0 + 0.5 * f)
    np.testing.assert_allclose(K.scaled_frequency(wave(100.0 / 3), s), wave(100.0 / 3))   # both ends of the ramp are continuous
    np.testing.assert_allclose(K.scaled_frequency(wave(100.0), s), wave(100.0) / 4.0)
    assert K.scaled_frequency(f, None) == f


def test_rotation_pairs_halves_and_depends_on_distance_only():
    rng = np.random.default_rng(1)
    q, k = rng.standard_normal(10), rng.standard_normal(10)
    s = {"factor": 2.0, "low": 1.0, "high": 2.0, "original": 40}
    d = lambda pq, pk: K.rotate_halves(q, pq, 6, 300.0, s) @ K.rotate_halves(k, pk, 6, 300.0, s)
    assert abs(d(17, 5) - d(112, 100)) < 1e-9 and abs(d(17, 5) - d(17, 6)) > 1e-6
    r = K.rotate_halves(q, 3, 6, 300.0)
    np.testing.assert_allclose([r[0], r[3]], [q[0] * np.cos(3.0) - q[3] * np.sin(3.0), q[3] * np.cos(3.0) + q[0] * np.sin(3.0)])
    assert np.allclose(r[6:], q[6:])


def test_sink_takes_mass_but_gives_nothing():
    s = np.array([0.3, -1.0, 2.0])
    np.testing.assert_allclose(K.sink_softmax(s, 1.0), np.exp(s) / (np.exp(s).sum() + np.e))
    np.testing.assert_allclose(K.sink_softmax(s, -1e9).sum(), 1.0)


def test_sum_norm_and_clamped_gate():
    x, y, w = np.array([1.0, -2.0, 0.5]), np.array([0.3, 0.1, -1.0]), np.array([1.0, 2.0, -1.0])
    s = 1.5 * x + y
    np.testing.assert_allclose(K.sum_norm(x, y, 1.5, w, 1e-3), s / np.sqrt((s * s).mean() + 1e-3) * w)
    sg = lambda t: 1 / (1 + math.exp(-1.702 * t))
    got = K.glu(np.array([5.0, -5.0, 0.4]), np.array([9.0, -9.0, 0.2]), 2.0)
    np.testing.assert_allclose(got, [2.0 * sg(2.0) * 3.0, -5.0 * sg(-5.0) * -1.0, 0.4 * sg(0.4) * 1.2])   # the gate has no lower clamp


def test_delta_rule_reads_its_own_write_and_forgets_by_the_head():
    k, v = np.array([0.6, 0.8]), np.array([2.0, -1.0, 3.0])
    S, o = K.delta_rule(np.zeros((2, 3)), k, k, v, 1.0, 0.3)
    np.testing.assert_allclose(o, v)                                             # unit key, beta 1: read back what was just written
    S, o = K.delta_rule(S, k, np.array([1.0, 0.0]), np.zeros(3), 0.0, 0.25)      # beta 0: only the decay acts
    np.testing.assert_allclose(o, 0.25 * v); np.testing.assert_allclose(S, 0.25 * np.outer(k, v))
    S2, _ = K.delta_rule(S, k, k, v, 1.0, 1.0)                                   # the old value under this key is replaced, not added to
    np.testing.assert_allclose(S2.T @ k, v)


def test_gla_decay_acts_on_key_channels():
    S = np.ones((2, 3))
    S, o = K.gla_rule(S, np.array([1.0, 0.0]), np.array([0.0, 1.0]), np.array([5.0, 6.0, 7.0]), np.array([0.5, 0.25]))
    np.testing.assert_allclose(S, [[0.5] * 3, [5.25, 6.25, 7.25]]); np.testing.assert_allclose(o, [0.5] * 3)
    np.testing.assert_allclose(K.channel_decay(np.array([0.0]), 16.0), [0.5 ** (1 / 16)])


def test_short_convolution_ends_at_the_current_token():
    w = np.array([[1.0, 10.0, 100.0]])
    y0, h = K.short_conv(w, np.zeros((2, 1)), np.array([3.0]))
    y1, h = K.short_conv(w, h, np.array([5.0]))
    y2, _ = K.short_conv(w, h, np.array([7.0]))
    assert (y0[0], y1[0], y2[0]) == (300.0, 530.0, 753.0)


def test_values_are_mixed_with_the_first_mixing_layers_own_values():
    rng = np.random.default_rng(4)
    cfg = K.make_config([("attention", K.attention_mixer(), None), ("attention", K.attention_mixer(v_mix=True), None),
                         ("attention", K.attention_mixer(v_mix=True), None), ("attention", K.attention_mixer(), None)])
    w = K.random_weights(cfg, rng)
    toks = rng.integers(0, cfg["vocab"], 9).tolist()
    base = K.run_sequence(cfg, w, toks)
    differs = lambda **ch: np.abs(K.run_sequence(cfg, {**w, **{k.replace("_", "."): v for k, v in ch.items()}}, toks) - base).max() > 1e-6
    assert not differs(l1_mix_vmix=np.asarray(0.9)) and differs(l2_mix_vmix=np.asarray(0.9))   # the first one's own weight is unused
    w1 = dict(w); w1["l2.mix.vmix"] = np.asarray(1.0)
    a = K.run_sequence(cfg, w1, toks)
    w1["l2.mix.v"] = w["l2.mix.v"] * -3.0                                        # lambda 1: layer 2's own values no longer matter
    np.testing.assert_allclose(K.run_sequence(cfg, w1, toks), a)
    assert "l0.mix.vmix" not in w and "l3.mix.vmix" not in w


def test_far_tokens_matter_only_through_what_keeps_them():
    """Attention alone: a token neither kept nor in the window is gone; the recurrent mixers remember."""
    rng = np.random.default_rng(5)
    att = K.make_config([("attention", K.attention_mixer(size=4, keep_first=2), K.dense_mlp(8))])
    w = K.random_weights(att, rng)
    toks = rng.integers(0, 80, 14).tolist()
    swap = lambda t, i: t[:i] + [(t[i] + 1) % 80] + t[i + 1:]
    base = K.run_sequence(att, w, toks)
    assert np.abs(K.run_sequence(att, w, swap(toks, 1))[13] - base[13]).max() > 1e-6       # kept
    moved = np.abs(K.run_sequence(att, w, swap(toks, 5)) - base).max(-1)
    assert moved[8] > 1e-6 and moved[9:].max() < 1e-12                                     # seen from 5 .. 8 only
    for mix in (("delta", K.delta_mixer()), ("gla", K.gla_mixer())):
        cfg = K.make_config([(mix[0], mix[1], None)])
        w = K.random_weights(cfg, rng)
        assert np.abs(K.run_sequence(cfg, w, swap(toks, 0))[13] - K.run_sequence(cfg, w, toks)[13]).max() > 1e-9


# ------------------------------------------------------------------------------------------------ registry, scheduler

def test_model_registry_reads_config_json():
    from nano_vllm_rs_b200.engine import Config, lib
    assert b"Kalesun" in lib().nvllm_registered_architectures()
    c = Config(model_config=json.dumps(small_cfg(vocab=77, width=24)))
    assert (c.arch, c.vocab_size, c.hidden_size, c.num_hidden_layers, c.recurrent_state) == ("Kalesun", 77, 24, 4, 1)
    only = K.make_config([("attention", K.attention_mixer(), K.dense_mlp(10))])
    assert Config(model_config=json.dumps(only)).recurrent_state == 0          # attention alone holds nothing but pages


@pytest.mark.parametrize("breakage,needle", [
    (lambda c: c["layers"][0].update(type="linear"), "linear"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "heads"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=3), "rot dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "rot dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("high"), "high"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(low=9.0), "scaling"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=7), "same kv_heads and vdim"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][2]["mixer"].update(conv=17), "conv"),
    (lambda c: c["layers"][0]["mixer"].pop("tau"), "tau"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "sparse"),
    (lambda c: c.pop("postln_alpha"), "postln_alpha"),
])
def test_bad_model_configs_are_refused_with_a_reason(breakage, needle):
    from nano_vllm_rs_b200 import _ffi
    from nano_vllm_rs_b200.engine import Config
    cfg = small_cfg()
    breakage(cfg)
    with pytest.raises(_ffi.NvllmError) as e:
        Config(model_config=json.dumps(cfg))
    assert needle in str(e.value)


def test_portion_steps_take_pages_and_slots_and_return_both():
    from nano_vllm_rs_b200.engine import Config, SamplingParams, Scheduler
    cfg = Config(model_config=json.dumps(small_cfg()), kvcache_block_size=16, num_kvcache_blocks=4, max_num_seqs=2,
                 max_num_batched_tokens=64, max_model_len=64)
    s = Scheduler(cfg)
    sp = SamplingParams(temperature=0.0, max_tokens=1, ignore_eos=True)
    a, b = s.add_sequence(list(range(20)), sp), s.add_sequence(list(range(30)), sp)
    s.schedule_chunks([a, b], [17, 2]); s.commit_chunks()
    s.schedule_chunks([a, b], [3, 28]); s.commit_chunks()           # the pool of pages and both slots are in use
    s.finish_sequence(a); s.release_sequence(a)
    c = s.add_sequence(list(range(32)), sp)
    batch = s.schedule_chunks([c], [32])
    assert len(set((np.asarray(batch.slot_mapping) // 16).tolist())) == 2
