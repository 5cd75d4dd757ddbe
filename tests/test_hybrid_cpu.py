"""Layer-list decoders without a GPU: configuration and weight loading, state slots and fed steps of the
scheduler, and the whole engine on the CPU backend against the plain implementation."""
import io
import json

import numpy as np
import pytest

import hybrid_models as hm
import hybrid_oracle as oracle
from oxide_tech_llm_engine_b200._build import host_ext
from oxide_tech_llm_engine_b200.errors import ConfigError, EngineError, ModelLoadError
from oxide_tech_llm_engine_b200.models.config import preset
from oxide_tech_llm_engine_b200.models.layer_spec import kipolix_config, kipolix_json, layer_runs
from oxide_tech_llm_engine_b200.models.registry import architecture, config_from_json
from oxide_tech_llm_engine_b200.models.weights import SyntheticSource, open_weights
from oxide_tech_llm_engine_b200.sampling_params import SamplingParams


def toks(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


# ---------------------------------------------------------------- configuration, registry, weights
def test_configuration_round_trips_and_reaches_the_registry():
    for c in hm.CONFIGS.values():
        mc = config_from_json(c)
        assert kipolix_json(mc) == c and mc.arch == "kipolix"
        assert architecture(mc).name == "kipolix" and architecture(preset("tiny")).name == "llama"
        assert mc.n_params() == sum(int(np.prod(x.shape)) for x in hm.weights(c).values())
    assert layer_runs(5, (1, 3, 3)) == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert config_from_json({"num_attention_heads": 8}) is None      # a Hugging Face configuration
    with pytest.raises(ConfigError):
        config_from_json({"architecture": "Unheard"})
    bad = json.loads(json.dumps(hm.CONFIGS["mixed"]))
    bad["layers"][0]["type"] = "convolution"
    with pytest.raises(ConfigError):
        kipolix_config(bad)


def test_weights_load_from_a_model_folder(tmp_path):
    c = hm.CONFIGS["mixed"]
    w = hm.weights(c, 3)
    hm.write_model(tmp_path / "m", c, w)
    src = open_weights(str(tmp_path / "m"))
    assert src.cfg == kipolix_config(c) and src.cfg.is_recurrent
    for n, x in w.items():
        assert np.array_equal(src.f32(n), x), n
    w2 = dict(w)
    w2["l1.mix.q"] = w2["l1.mix.q"][:-1]
    hm.write_model(tmp_path / "bad", c, w2)
    with pytest.raises(ModelLoadError):
        open_weights(str(tmp_path / "bad"))


# ---------------------------------------------------------------- scheduler
def mk_sched(slots=2, blocks=16, seqs=2, **kw):
    H = host_ext()
    sc = H.SchedulerConfig()
    sc.num_blocks, sc.max_num_seqs, sc.max_num_batched_tokens, sc.max_blocks_per_seq = blocks, seqs, 64, blocks
    sc.chunk_min, sc.chunk_max, sc.sla_budget, sc.state_slots = 8, 64, False, slots
    for k, v in kw.items():
        setattr(sc, k, v)
    return H.Scheduler(sc)


def test_scheduler_gives_every_running_sequence_a_state_slot_and_takes_it_back():
    s = mk_sched()
    for i in range(3):
        s.add_request(i, np.arange(5 + i, dtype=np.int32), 3, [], True)
    p = s.schedule()
    assert sorted(p.prefill_slots.tolist()) == [0, 1] and s.num_free_slots() == 0 and s.num_waiting() == 1
    first = dict(zip(p.prefill_ids.tolist(), p.prefill_slots.tolist()))
    assert p.prev_ids.tolist() == [-1, 0, 1, 2, 3, -1, 0, 1, 2, 3, 4]
    s.update(p, np.array([50, 51], dtype=np.int32))
    p = s.schedule()
    assert dict(zip(p.decode_ids.tolist(), p.decode_slots.tolist())) == first     # a sequence keeps its slot
    assert p.token_ids.tolist() == [50, 51] and p.prev_ids.tolist() == [4, 5]
    s.update(p, np.array([52, 53], dtype=np.int32))
    ok, _ = s.cancel(0)
    assert ok and s.num_free_slots() == 1
    p = s.schedule()                                                               # the waiting one is admitted
    assert p.prefill_ids.tolist() == [2] and p.prefill_slots.tolist() == [first[0]]
    while s.has_work():
        s.update(p, np.zeros(p.logit_rows.size, dtype=np.int32))
        p = s.schedule()
    assert s.num_free_slots() == 2 and s.num_free_blocks() == 16


def test_preemption_returns_the_slot_and_restarts_from_the_first_token():
    s = mk_sched(blocks=5, seqs=2)
    for i in range(2):
        s.add_request(i, np.arange(30, dtype=np.int32), 20, [], True)
    seen = set()
    for _ in range(200):
        if not s.has_work():
            break
        p = s.schedule()
        for rid, start, n, slot in zip(p.prefill_ids, p.q_start, p.q_lens, p.prefill_slots):
            if p.positions[start] == 0:
                assert p.prev_ids[start] == -1 and slot >= 0
                seen.add((int(rid), int(n)))
        s.update(p, np.ones(p.logit_rows.size, dtype=np.int32))
    assert s.preemptions() >= 1 and any(n > 30 for _, n in seen)   # recomputed with its generated tokens
    assert s.num_free_slots() == 2 and s.num_free_blocks() == 5


def test_recurrent_state_rules_out_drafts_prefix_reuse_and_pruning():
    s = mk_sched(enable_radix=True)
    s.add_request(0, np.arange(40, dtype=np.int32), 8, [], True)
    s.update(s.schedule(), np.array([1], dtype=np.int32))
    s.set_drafts(0, [1, 2])
    p = s.schedule()
    assert p.n_decode == 1 and p.n_tokens == 1 and s.prune_request(0, [], 1, 1, 1) == []
    s.update(p, np.array([2], dtype=np.int32))
    s.cancel(0)
    s.add_request(1, np.arange(40, dtype=np.int32), 8, [], True)
    assert s.schedule().n_tokens == 40


def test_fed_steps_batch_single_tokens_beside_chunks():
    s = mk_sched(slots=3, seqs=3)
    p = s.feed([(7, [1, 2, 3], [0, 2]), (8, [9], [0])])
    assert p.n_decode == 0 and p.q_lens.tolist() == [3, 1] and p.logit_rows.tolist() == [0, 2, 3]
    s.feed_done(p)
    p = s.feed([(7, [4, 5], [1]), (8, [10], [0]), (9, list(range(20)), [])])
    assert p.decode_ids.tolist() == [8] and p.token_ids.tolist()[:3] == [10, 4, 5]
    assert p.prev_ids.tolist()[:4] == [9, 3, 4, -1] and p.positions.tolist()[:3] == [1, 3, 4]
    assert p.logit_rows.tolist() == [2, 0] and p.logit_req.tolist() == [7, 8]      # order of the entries
    s.feed_done(p)
    with pytest.raises(ValueError):
        s.add_request(1, np.arange(3, dtype=np.int32), 1, [], True)
    with pytest.raises(ValueError):
        s.feed([(7, [1], [1])])
    with pytest.raises(RuntimeError):
        s.feed([(11, [1], [])])           # a fourth live request
    for i in (7, 8, 9):
        s.cancel(i)
    assert s.num_free_blocks() == 16 and s.num_free_slots() == 3
    s.add_request(1, np.arange(3, dtype=np.int32), 1, [], True)
    with pytest.raises(ValueError):
        s.feed([(7, [1], [])])


# ---------------------------------------------------------------- the plain implementation is sharp
def test_the_test_models_show_every_mistake(monkeypatch):
    """A planted mistake in the plain implementation moves the logits by far more than the tolerances."""
    c = hm.CONFIGS["mixed"]
    w, t = hm.weights(c, 1), toks(110, 300, 5)
    good = oracle.forward(c, w, t).numpy()

    def changed(cfg=c, tokens=t, patch=None):
        with pytest.MonkeyPatch.context() as mp:
            for name, fn in (patch or {}).items():
                mp.setattr(oracle, name, fn)
            return hm.error(oracle.forward(cfg, w, tokens).numpy(), good)

    def cfg(fn):
        x = json.loads(json.dumps(c))
        fn(x)
        return x

    mask = lambda k, d: cfg(lambda x: x["layers"][1]["mixer"]["mask"].__setitem__(k, x["layers"][1]["mixer"]["mask"][k] + d))
    rot, keep = oracle.rotate, oracle.embedding
    cases = {
        "window +1": changed(mask("size", 1)), "window -1": changed(mask("size", -1)),
        "kept +1": changed(mask("keep_first", 1)), "kept -1": changed(mask("keep_first", -1)),
        "layout": changed(patch={"rotate": lambda x, p, b, d, i: rot(x, p, b, d, not i)}),
        "position +1 of keys": changed(patch={"rotate": lambda x, p, b, d, i: rot(x, p + (x.shape[1] == 3), b, d, i)}),
        "decay": changed(cfg(lambda x: x["layers"][0]["mixer"].update(decay=[0.9, 0.98, 0.995]))),
        "loop": changed(cfg(lambda x: x["loop"].update(times=3))),
        "bigram": changed(cfg(lambda x: x["embedding"]["bigram"].update(mul_prev=8))),
        "first row": changed(patch={"embedding": lambda c_, w_, t_: keep(
            c_, {**w_, "bigram": w_["bigram"].clone().index_fill_(0, oracle.torch.tensor(61), 0.0)}, t_)}),
        "eps": changed(cfg(lambda x: x["norm"].update(eps=1e-2))),
    }
    assert all(v > 0.05 for v in cases.values()), cases


# ---------------------------------------------------------------- engine on the CPU backend
@pytest.mark.parametrize("name", list(hm.CONFIGS))
def test_cpu_engine_equals_the_plain_implementation(name):
    c = hm.CONFIGS[name]
    w = hm.weights(c, 2)
    eng = hm.engine(c, w, backend="cpu", live=2, blocks=24)
    seqs = [toks(n, c["vocab"], n) for n in (1, 45, 90, 2, 33, 64)]
    want = [oracle.forward(c, w, t).numpy() for t in seqs]
    for t, x in zip(seqs, want):
        assert hm.error(hm.feed_all(eng, 0, t, []), x) < 1e-4
        assert hm.error(hm.feed_all(eng, 0, t, [2, 3, 1, 1, 17, 2]), x) < 1e-4
    for got, x in zip(hm.interleaved(eng, seqs, 11), want):
        assert hm.error(got, x) < 1e-4
    assert eng.sched.num_free_blocks() == 24


@pytest.mark.parametrize("name", ["mixed", "attention", "retention"])
def test_cpu_generation_through_the_scheduler_is_greedy_decoding(name):
    c = hm.CONFIGS[name]
    w = hm.weights(c, 4)
    # a pool that is short for three sequences at once: chunked prompts, preemption, slots used again
    eng = hm.engine(c, w, backend="cpu", live=3, blocks=9, tokens=24, chunk_min=4, chunk_max=24, sla_budget=False,
                    speculative="ngram", enable_radix=True)
    assert (eng._drafter is None) == (name != "attention")
    prompts = [toks(n, c["vocab"], 70 + n) for n in (3, 50, 41, 17, 1)]
    outs = eng.generate(prompts, SamplingParams(greedy=True, max_tokens=24, ignore_eos=True))
    for p, o in zip(prompts, outs):
        lg = oracle.forward(c, w, p + o[:-1]).numpy()[len(p) - 1:]
        assert len(o) == 24 and (lg.argmax(-1) == np.array(o)).all()
    assert name != "mixed" or eng.sched.preemptions() > 0


def test_refused_options_and_formats(tmp_path):
    c = hm.CONFIGS["mixed"]
    w = hm.weights(c, 0)
    for kw in (dict(h2o_pruning=True), dict(context_shift=True), dict(comm="nccl")):
        with pytest.raises(ConfigError):
            hm.engine(c, w, backend="cpu", **kw)
    from oxide_tech_llm_engine_b200.engine.cskv import save_sequence

    eng = hm.engine(c, w, backend="cpu")
    eng.feed([(0, [1, 2], [])])
    with pytest.raises(EngineError):
        save_sequence(eng, 0, str(tmp_path / "x"))


def test_command_line_serves_a_preset_and_a_model_folder(tmp_path, capsys):
    from oxide_tech_llm_engine_b200 import cli

    c = hm.model(64, 256, [hm.mlp(hm.att(2, 1, 32, 32, 16, 20, 2), 64), hm.mlp(hm.ret(2, 16, 16, 16, [0.9, 0.99]), 64)])
    hm.write_model(tmp_path / "m", c, hm.weights(c, 1))
    for m in (str(tmp_path / "m"), "kipolix-tiny"):
        assert cli.main(["verify", "-m", m, "-b", "cpu", "--greedy", "-c", "256", "--max-slots", "2"]) == 0
        out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
        assert len(out["tokens"]) == 16


def test_trace_replay_writes_the_wanted_logits_in_order(tmp_path, capsys):
    from oxide_tech_llm_engine_b200.trace_run import Replay, build_engine

    c = hm.CONFIGS["attention"]
    w = hm.weights(c, 6)
    hm.write_model(tmp_path / "m", c, w)
    a, b = toks(40, 130, 1), toks(9, 130, 2)
    want_a, want_b = oracle.forward(c, w, a).numpy(), oracle.forward(c, w, b).numpy()
    r = Replay(build_engine(str(tmp_path / "m"), "bfloat16", 64, backend="cpu"))
    got = r.step({"step": 0, "entries": [{"id": "x", "tokens": a[:30], "want": [29, 3, 3]}], "end": []})
    assert hm.error(got, want_a[[29, 3, 3]]) < 1e-4
    got = r.step({"step": 1, "entries": [{"id": "y", "tokens": b, "want": []}, {"id": "x", "tokens": a[30:31], "want": [0]}],
                  "end": ["y"]})
    assert got.shape == (1, 130) and hm.error(got, want_a[[30]]) < 1e-4
    got = r.step({"step": 2, "entries": [{"id": "y", "tokens": b, "want": [8]}, {"id": "x", "tokens": a[31:], "want": [8]}],
                  "end": ["x", "y"]})
    assert hm.error(got, np.stack([want_b[8], want_a[39]])) < 1e-4
    assert r.step({"step": 3, "entries": [], "end": []}).shape == (0, 130)
    assert r.engine.sched.num_free_blocks() == 4 and not r.ids


def test_synthetic_weights_start_as_a_plain_residual():
    src = SyntheticSource(preset("kipolix-tiny"), seed=1)
    assert np.array_equal(src.f32("l0.hc1.mix"), np.eye(2)) and np.all(src.f32("l0.norm1") == 0)
    assert np.all(src.f32("l0.mix.q.norm") == 1) and src.f32("bigram").shape == (1001, 128)
