"""Vokepel models without a GPU: configuration, weights, the plain implementation's sharpness, and the whole engine on the CPU
backend against it."""
import json

import numpy as np
import pytest
import torch

import hybrid_models as hm
import vokepel_models as vm
import vokepel_oracle as oracle
from oxide_tech_llm_engine_b200.errors import ConfigError, ModelLoadError
from oxide_tech_llm_engine_b200.models.config import preset
from oxide_tech_llm_engine_b200.models.layer_spec import vokepel_config, vokepel_json
from oxide_tech_llm_engine_b200.models.registry import architecture, config_from_json
from oxide_tech_llm_engine_b200.models.weights import SyntheticSource, open_weights, tensor_names
from oxide_tech_llm_engine_b200.sampling_params import SamplingParams
from test_zagolix_cpu import changed, setting, toks


# ---------------------------------------------------------------- configuration and weights
def test_configuration_round_trips_and_reaches_the_registry():
    for name, c in vm.CONFIGS.items():
        mc = config_from_json(c)
        assert vokepel_json(mc) == c and mc.arch == "vokepel" and architecture(mc).name == "vokepel" and mc.tie_embeddings
        assert mc.is_recurrent == (name != "talk")
        assert mc.n_params() == mc.active_params() == sum(int(np.prod(x.shape)) for x in vm.weights(c).values())
    mc = vokepel_config(vm.CONFIGS["mixed"])
    assert mc.layer_runs == [0, 1, 2, 1, 2, 3] and mc.pass_starts == {1: 0, 3: 1}
    # keys that are values are kept once; a looped layer keeps something in every pass
    assert mc.kv_bytes_per_token() == 2 * (3 * 80 + 2 * 40 + 2 * (80 + 96) + 3 * 72)
    bad = [("layers", 0, "type", "ssd"), ("layers", 1, "mixer", "vdim", 41), ("layers", 3, "mixer", "kv_heads", 4), ("layers", 1, "mlp", "kind", "moe"),
           ("layers", 0, "mixer", "left", "kv_heads", 4), ("layers", 0, "mixer", "left", "rot", {"base": 10.0, "dims": 50}), ("loop", "stop", 5),
           ("loop", "times", 0)]
    for b in bad:
        with pytest.raises(ConfigError):
            vokepel_config(changed(vm.CONFIGS["mixed"], setting(*b)))


def test_weights_load_from_a_model_folder(tmp_path):
    c = vm.CONFIGS["mixed"]
    w = vm.weights(c, 3)
    assert w["loop.in"].shape == (160, 320) and w["loop.step"].shape == (2, 160) and "head" not in w and "l2.norm2" not in w and "l1.mix.v" not in w
    assert "loop.in" not in vm.weights(vm.CONFIGS["talk"])
    hm.write_model(tmp_path / "m", c, w)
    src = open_weights(str(tmp_path / "m"))
    assert src.cfg == vokepel_config(c)
    for n, x in w.items():
        assert np.array_equal(src.f32(n), x), n
    for bad in ("loop.step", "l1.mix.talk", "l0.mix.left.sink", "l2.mix.right.z.b", "l0.mlp.up"):
        w2 = dict(w)
        w2[bad] = w2[bad][:-1]
        hm.write_model(tmp_path / "bad", c, w2)
        with pytest.raises(ModelLoadError):
            open_weights(str(tmp_path / "bad"))


def test_synthetic_weights_start_with_heads_of_their_own_and_open_states():
    mc = preset("vokepel-tiny")
    src = SyntheticSource(mc, seed=1)
    assert np.abs(src.f32("l1.mix.talk") - np.eye(3)).max() < 0.2 and src.f32("l0.mix.right.z.b").max() <= -1 and src.f32("l1.mix.r1").min() > 0
    assert np.abs(src.f32("loop.in")[:, :128] - np.eye(128)).max() < 0.2 and {n for n, _ in tensor_names(mc)} == set(src.names())


# ---------------------------------------------------------------- the plain implementation is sharp
def test_the_test_models_show_every_mistake():
    """A planted mistake in the plain implementation moves the logits by far more than the tolerances."""
    c = vm.CONFIGS["mixed"]
    w, t = vm.weights(c, 1), toks(150, 300, 5)
    good = oracle.forward(c, w, t).numpy()

    def off(cfg=None, weights=w, **patch):
        with pytest.MonkeyPatch.context() as mp:
            for name, fn in patch.items():
                mp.setattr(oracle, name, fn)
            return hm.error(oracle.forward(changed(c, setting(*cfg)) if cfg else c, weights, t).numpy(), good)

    o = oracle
    softmax, talk, scores, cap, bias, gru, rotate, enter, cand = (o.masked_softmax, o.talk, o.raw_scores, o.cap, o.distance_bias, o.gru, o.rotate,
                                                                  o.enter_pass, o.candidate)

    def normed_values(cf, z, p, h, pos, eps):
        with pytest.MonkeyPatch.context() as mp:
            k = (o.rms(h @ z[p + "k"].T, eps) * z[p + "k.norm"]).view(len(h), cf["kv_heads"], cf["dim"])
            mp.setattr(o, "values_of", lambda a, v, keep=o.values_of: keep(a, k))
            return o.mix_attention(cf, z, p, h, pos, eps)

    state_of_one_chunk = lambda z, x: torch.cat([gru(z[:64], x[:64]), gru(z[64:], x[64:])])
    swap = lambda a, b: {**w, a: w[b], b: w[a]}
    half = lambda x, p, b, d, i: rotate(x, p, b, d, False)
    cases = {
        "window out": off(masked_softmax=lambda s, n, k=None: softmax(s, n + 1, k)), "window in": off(masked_softmax=lambda s, n, k=None: softmax(s, n - 1, k)),
        "no sink": off(masked_softmax=lambda s, n, k=None: softmax(s, n)),
        "sinks of other heads": off(masked_softmax=lambda s, n, k=None: softmax(s, n, None if k is None else k.flip(0))),
        "sink scaled": off(masked_softmax=lambda s, n, k=None: softmax(s, n, None if k is None else 0.3 * k)),
        "talk transposed": off(talk=lambda s, m: talk(s, m.T)), "no talk": off(talk=lambda s, m: s),
        "talk before the cap": off(cap=lambda s, n: s, talk=lambda s, m: cap(talk(s, m), 12.0)),
        "no cap": off(cap=lambda s, n: s), "cap": off(("layers", 3, "mixer", "softcap", 12.0)), "other cap": off(("layers", 1, "mixer", "softcap", 9.0)),
        "bias one further": off(distance_bias=lambda n, a, b: a[:, None, None] * torch.log(1 + b[:, None, None] * ((torch.arange(n)[:, None] - torch.arange(n)).clamp(min=0) + 1))),
        "no bias": off(distance_bias=lambda n, a, b: 0 * bias(n, a, b)), "bias rates": off(distance_bias=lambda n, a, b: bias(n, b, a.abs())),
        "values normed": off(MIXERS={**o.MIXERS, "attention": normed_values}),
        "no gate": off(weights={**w, **{n: 0 * x for n, x in w.items() if n in ("l1.mix.g", "l3.mix.g")}}),
        "gate of silu": off(sigmoid=lambda z: z / (1 + torch.exp(-z))),
        "a key ahead": off(raw_scores=lambda q, k, s: scores(q, k.roll(1, 0), s)),
        "rotation of the halves": off(rotate=half), "base": off(("layers", 0, "mixer", "left", "rot", "base", 1500.0)),
        "rotated one further": off(rotate=lambda x, p, b, d, i: rotate(x, p + p, b, d, i)),
        "state lost": off(gru=state_of_one_chunk), "gates swapped": off(gru=lambda z, x: gru(1 - z, x)), "candidate": off(candidate=lambda u: u),
        "left scale": off(("layers", 0, "mixer", "left_scale", 1.0)), "right scale": off(("layers", 2, "mixer", "right_scale", 1.0)),
        "squared": off(MIXERS=o.MIXERS, feed_forward=lambda z, p, h: torch.relu(h @ z[p + "up"].T) @ z[p + "down"].T),
        "residual": off(("residual_mult", 1.0)), "logit scale": off(("logit_scale", 0.5)), "logit cap": off(("logit_softcap", 12.0)),
        "no entry": off(enter_pass=lambda x, x0, z, k: x), "entry of the embedding twice": off(enter_pass=lambda x, x0, z, k: enter(x0, x0, z, k)),
        "entry the other way": off(enter_pass=lambda x, x0, z, k: enter(x0, x, z, k)), "first step twice": off(enter_pass=lambda x, x0, z, k: enter(x, x0, z, 0)),
        "passes": off(weights={**w, "loop.step": np.concatenate([w["loop.step"], w["loop.step"][:1]])}, cfg=("loop", "times", 3)),
        "norms swapped": off(weights=swap("l0.norm1", "l0.norm2")), "head norm weights": off(weights={**w, "l1.mix.k.norm": 0 * w["l1.mix.k.norm"] + 1}),
        "eps": off(("norm", "eps", 3e-2)), "score scale": off(("layers", 1, "mixer", "scale", 0.2)),
    }
    assert all(v > 0.01 for v in cases.values()), {k: v for k, v in cases.items() if not v > 0.01}


def test_candidates_are_continuous_and_states_stay_between_them():
    u = torch.tensor([-1e-9, 0.0, 1e-9, -3.0, 4.0], dtype=torch.float64)
    assert torch.allclose(oracle.candidate(u), torch.tensor([0.5, 0.5, 0.5, 1 / (1 + np.exp(3.0)), 4.5], dtype=torch.float64))
    z, c = torch.rand(50, 7, dtype=torch.float64), torch.rand(50, 7, dtype=torch.float64) + 1.0
    s = oracle.gru(z, c)
    assert bool((s[1:] <= torch.maximum(s[:-1], c[1:]) + 1e-12).all()) and bool((s > 0).all())


# ---------------------------------------------------------------- engine on the CPU backend
@pytest.mark.parametrize("name", list(vm.CONFIGS))
def test_cpu_engine_equals_the_plain_implementation(name):
    c = vm.CONFIGS[name]
    w = vm.weights(c, 2)
    eng = hm.engine(c, w, backend="cpu", live=2, blocks=24)
    seqs = [toks(n, c["vocab"], n) for n in (1, 45, 90, 2, 33)]
    want = [oracle.forward(c, w, t).numpy() for t in seqs]
    for t, x in zip(seqs, want):
        assert hm.error(hm.feed_all(eng, 0, t, []), x) < 1e-4
        assert hm.error(hm.feed_all(eng, 0, t, [2, 3, 1, 1, 17, 2]), x) < 1e-4
    for got, x in zip(hm.interleaved(eng, seqs, 11), want):
        assert hm.error(got, x) < 1e-4
    assert eng.sched.num_free_blocks() == 24 and (name == "talk" or eng.sched.num_free_slots() == 2)


def test_cpu_generation_through_the_scheduler_is_greedy_decoding():
    c = vm.CONFIGS["mixed"]
    w = vm.weights(c, 4)
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


def test_prefix_cache_shares_keys_and_their_norms_of_models_without_state():
    c = vm.CONFIGS["talk"]
    w = vm.weights(c, 4)
    eng = hm.engine(c, w, backend="cpu", live=2, blocks=24, enable_radix=True)
    head = toks(64, 200, 1)
    for tail in ([], [5, 6, 7], toks(20, 200, 2)):
        p = head + tail
        o = eng.generate([p], SamplingParams(greedy=True, max_tokens=6, ignore_eos=True))[0]
        lg = oracle.forward(c, w, p + o[:-1]).numpy()[len(p) - 1:]
        assert (lg.argmax(-1) == np.array(o)).all()
    assert eng.stats["prefill_tokens"] < 64 + 67 + 84          # the second and third prompt found the first one's blocks


def test_command_line_serves_a_preset_and_a_model_folder(tmp_path, capsys):
    from oxide_tech_llm_engine_b200 import cli

    c = vm.model(64, 256, [vm.mlp(vm.talk(2, 1, 16, 32), 48), vm.mlp(vm.pair(2, 1, 16, 24, 8, 40, 32), 40)], loop=(0, 2, 2))
    hm.write_model(tmp_path / "m", c, vm.weights(c, 1))
    for m in (str(tmp_path / "m"), "vokepel-tiny"):
        assert cli.main(["verify", "-m", m, "-b", "cpu", "--greedy", "-c", "256", "--max-slots", "2"]) == 0
        assert len(json.loads(capsys.readouterr().out.strip().splitlines()[-1])["tokens"]) == 16


def test_refused_options():
    c = vm.CONFIGS["ones"]
    for kw in (dict(h2o_pruning=True), dict(context_shift=True), dict(comm="nccl")):
        with pytest.raises(ConfigError):
            hm.engine(c, vm.weights(c), backend="cpu", **kw)


def test_passes_over_prompt_tiles_are_about_equal():
    from oxide_tech_llm_engine_b200.models import hybrid

    for n in (1, 5, 64, 301):
        for scores in (1000, 10 ** 7, 10 ** 9, 10 ** 10):
            step = hybrid.talk_pass(n, scores)
            assert 1 <= step <= n and (step == 1 or step * scores * 4 <= hybrid.TALK_SCORE_BYTES)
            passes = -(-n // step)
            assert n - (passes - 1) * step > step - passes
