"""Povatar models without a GPU: configuration, weights, the plain implementation's sharpness, and the whole engine
on the CPU backend against it."""
import json

import numpy as np
import pytest
import torch

import hybrid_models as hm
import povatar_models as pm
import povatar_oracle as oracle
from oxide_tech_llm_engine_b200.errors import ConfigError, ModelLoadError
from oxide_tech_llm_engine_b200.models.config import preset
from oxide_tech_llm_engine_b200.models.layer_spec import RotarySpec, YarnSpec, povatar_config, povatar_json
from oxide_tech_llm_engine_b200.models.registry import architecture, config_from_json
from oxide_tech_llm_engine_b200.models.weights import SyntheticSource, open_weights, tensor_names
from oxide_tech_llm_engine_b200.sampling_params import SamplingParams


def toks(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


def changed(cfg, fn):
    c = json.loads(json.dumps(cfg))
    fn(c)
    return c


# ---------------------------------------------------------------- configuration and weights
def test_configuration_round_trips_and_reaches_the_registry():
    for c in pm.CONFIGS.values():
        mc = config_from_json(c)
        assert povatar_json(mc) == c and mc.arch == "povatar" and architecture(mc).name == "povatar" and mc.is_recurrent
        assert mc.n_params() == sum(int(np.prod(x.shape)) for x in pm.weights(c).values())
    mc = povatar_config(pm.CONFIGS["mixed"])
    idle = 2 * 160 * ((7 - 3) * 40 + (33 - 1) * 100)
    assert mc.active_params() == mc.n_params() - idle
    assert mc.kv_bytes_per_token() == 2 * (3 * (48 + 32) + 80 + 96 + 4 * 128)
    for fn in (lambda c: c["layers"][0].update(type="serial"), lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4),
               lambda c: c["layers"][0]["mixer"]["right"].update(groups=4), lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=7),
               lambda c: c["layers"][0]["mlp"]["router"].update(top=8), lambda c: c["layers"][0]["mlp"].update(kind="dense")):
        with pytest.raises(ConfigError):
            povatar_config(changed(pm.CONFIGS["mixed"], fn))


def test_yarn_frequencies_equal_the_plain_ones():
    for dims, base, sc in ((24, 10000.0, (8.0, 64, 20.0, 1.0)), (64, 500.0, (2.0, 4096, 32.0, 1.0)), (8, 1e6, (40.0, 32768, 1.5, 1.0)),
                           (16, 300.0, (4.0, 3, 1.0, 0.9)), (10, 77.0, None)):
        spec = RotarySpec(dims, base, False, YarnSpec(*sc) if sc else None)
        f, gain = spec.frequencies()
        want, wg = oracle.yarn_frequencies(base, dims, dict(zip(("factor", "original", "fast", "slow"), sc)) if sc else None)
        assert np.allclose(f, want.numpy(), rtol=1e-14) and abs(gain - wg) < 1e-15


def test_weights_load_from_a_model_folder(tmp_path):
    c = pm.CONFIGS["mixed"]
    w = pm.weights(c, 3)
    hm.write_model(tmp_path / "m", c, w)
    src = open_weights(str(tmp_path / "m"))
    assert src.cfg == povatar_config(c)
    for n, x in w.items():
        assert np.array_equal(src.f32(n), x), n
    for bad in ("l0.mlp.e3.down", "l2.mix.right.conv"):
        w2 = dict(w)
        w2[bad] = w2[bad][:-1]
        hm.write_model(tmp_path / "bad", c, w2)
        with pytest.raises(ModelLoadError):
            open_weights(str(tmp_path / "bad"))


def test_synthetic_weights_have_sensible_time_constants():
    mc = preset("povatar-tiny")
    src = SyntheticSource(mc, seed=1)
    dt = np.log1p(np.exp(src.f32("l0.mix.right.dt_bias").astype(np.float64)))
    assert 0.0009 < dt.min() and dt.max() < 0.11 and np.all(src.f32("l0.norm2") == 1) and np.all(src.f32("l0.mix.right.D") == 1)
    assert {n for n, _ in tensor_names(mc)} == set(src.names())


# ---------------------------------------------------------------- the plain implementation is sharp
def test_the_test_models_show_every_mistake(monkeypatch):
    """A planted mistake in the plain implementation moves the logits by far more than the tolerances."""
    c = pm.CONFIGS["mixed"]
    w, t = pm.weights(c, 1), toks(150, 300, 5)
    good = oracle.forward(c, w, t).numpy()

    def off(cfg=c, weights=w, **patch):
        with pytest.MonkeyPatch.context() as mp:
            for name, fn in patch.items():
                mp.setattr(oracle, name, fn)
            return hm.error(oracle.forward(cfg, weights, t).numpy(), good)

    def cfg(layer, *path):
        def fn(x):
            at = x["layers"][layer]
            for k in path[:-2]:
                at = at[k]
            at[path[-2]] = path[-1]
        return changed(c, fn)

    L, R = ("mixer", "left"), ("mixer", "right")
    att, conv, ssd, gate, choose, half = (oracle.chunk_attention, oracle.short_conv, oracle.ssd, oracle.gated_group_norm, oracle.choose,
                                          oracle.rotate_half)
    w_swap = {**w, "l0.norm1": w["l0.norm2"], "l0.norm2": w["l0.norm1"]}
    cases = {
        "chunk +1": off(cfg(0, *L, "mask", "size", 38)), "chunk -1": off(cfg(0, *L, "mask", "size", 36)),
        "no sink": off(chunk_attention=lambda q, k, v, s, n: att(q, k, v, s, n, sink=False)),
        "no scaling": off(cfg(0, *L, "rot", "scaling", None)), "factor": off(cfg(0, *L, "rot", "scaling", "factor", 7.0)),
        "ramp": off(cfg(0, *L, "rot", "scaling", "fast", 3.0)),
        "rotation gain": off(rotate_half=lambda x, p, f, g: half(x, p, f, 1.0)),
        "position +1 of keys": off(rotate_half=lambda x, p, f, g: half(x, p + (x.shape[1] == 3), f, g)),
        "taps reversed": off(short_conv=lambda u, k, b: conv(u, k.flip(1), b)),
        "conv bias": off(short_conv=lambda u, k, b: conv(u, k, 0 * b)),
        "step clamp": off(ssd=lambda x, B, C, dt, A, D: ssd(x, B, C, dt.clamp(max=0.2), A, D)),
        "groups rolled": off(ssd=lambda x, B, C, dt, A, D: ssd(x, B.roll(1, 1), C, dt, A, D)),
        "no skip": off(ssd=lambda x, B, C, dt, A, D: ssd(x, B, C, dt, A, 0 * D)),
        "gate after norm": off(gated_group_norm=lambda y, z, k, n, e: oracle.rms(y.view(len(y), n, -1), e).reshape(y.shape) * k * oracle.silu(z)),
        "norm groups": off(cfg(0, *R, "norm_groups", 6)),
        "top": off(cfg(0, "mlp", "router", "top", 2)),
        "weights not divided": off(choose=lambda lg, k: (choose(lg, k)[0], torch.softmax(lg, -1).gather(1, choose(lg, k)[0]))),
        "relu": off(relu_squared=lambda z: z.clamp(min=0)),
        "norms swapped": off(weights=w_swap),
        "eps": off(changed(c, lambda x: x["norm"].update(eps=1e-2))), "scale": off(changed(c, lambda x: x["embedding"].update(scale=2.0))),
    }
    assert all(v > 0.02 for v in cases.values()), cases


# ---------------------------------------------------------------- engine on the CPU backend
@pytest.mark.parametrize("name", list(pm.CONFIGS))
def test_cpu_engine_equals_the_plain_implementation(name):
    c = pm.CONFIGS[name]
    w = pm.weights(c, 2)
    eng = hm.engine(c, w, backend="cpu", live=2, blocks=24)
    seqs = [toks(n, c["vocab"], n) for n in (1, 45, 90, 2, 33)]
    want = [oracle.forward(c, w, t).numpy() for t in seqs]
    for t, x in zip(seqs, want):
        assert hm.error(hm.feed_all(eng, 0, t, []), x) < 1e-4
        assert hm.error(hm.feed_all(eng, 0, t, [2, 3, 1, 1, 17, 2]), x) < 1e-4
    for got, x in zip(hm.interleaved(eng, seqs, 11), want):
        assert hm.error(got, x) < 1e-4
    assert eng.sched.num_free_blocks() == 24 and eng.sched.num_free_slots() == 2


def test_cpu_generation_through_the_scheduler_is_greedy_decoding():
    c = pm.CONFIGS["mixed"]
    w = pm.weights(c, 4)
    # a pool that is short for three sequences at once: chunked prompts, preemption, slots used again
    eng = hm.engine(c, w, backend="cpu", live=3, blocks=9, tokens=24, chunk_min=4, chunk_max=24, sla_budget=False, speculative="ngram",
                    enable_radix=True)
    assert eng._drafter is None
    prompts = [toks(n, 300, 70 + n) for n in (3, 50, 41, 17, 1)]
    outs = eng.generate(prompts, SamplingParams(greedy=True, max_tokens=20, ignore_eos=True))
    for p, o in zip(prompts, outs):
        lg = oracle.forward(c, w, p + o[:-1]).numpy()[len(p) - 1:]
        assert len(o) == 20 and (lg.argmax(-1) == np.array(o)).all()
    assert eng.sched.preemptions() > 0


def test_command_line_serves_a_preset_and_a_model_folder(tmp_path, capsys):
    from oxide_tech_llm_engine_b200 import cli

    c = pm.model(64, 256, [pm.layer(pm.left(2, 1, 32, 32, 24, (16, 1000.0)), pm.right(2, 16, 16, 1, 3, 2), (5, 2, 48))] * 2)
    hm.write_model(tmp_path / "m", c, pm.weights(c, 1))
    for m in (str(tmp_path / "m"), "povatar-tiny"):
        assert cli.main(["verify", "-m", m, "-b", "cpu", "--greedy", "-c", "256", "--max-slots", "2"]) == 0
        assert len(json.loads(capsys.readouterr().out.strip().splitlines()[-1])["tokens"]) == 16


def test_refused_options():
    c = pm.CONFIGS["ones"]
    for kw in (dict(h2o_pruning=True), dict(context_shift=True), dict(comm="nccl")):
        with pytest.raises(ConfigError):
            hm.engine(c, pm.weights(c), backend="cpu", **kw)
