"""Zagolix models without a GPU: configuration, weights, the plain implementation's sharpness, and the whole engine on the
CPU backend against it."""
import json

import numpy as np
import pytest
import torch

import hybrid_models as hm
import zagolix_models as zm
import zagolix_oracle as oracle
from oxide_tech_llm_engine_b200.errors import ConfigError, ModelLoadError
from oxide_tech_llm_engine_b200.models.config import preset
from oxide_tech_llm_engine_b200.models.layer_spec import zagolix_config, zagolix_json
from oxide_tech_llm_engine_b200.models.registry import architecture, config_from_json
from oxide_tech_llm_engine_b200.models.weights import SyntheticSource, open_weights, tensor_names
from oxide_tech_llm_engine_b200.sampling_params import SamplingParams


def toks(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


def changed(cfg, fn):
    c = json.loads(json.dumps(cfg))
    fn(c)
    return c


def setting(*path):
    """A change of a configuration: keys, the last of them the new value."""
    def fn(c):
        for k in path[:-2]:
            c = c[k]
        c[path[-2]] = path[-1]
    return fn


# ---------------------------------------------------------------- configuration and weights
def test_configuration_round_trips_and_reaches_the_registry():
    for name, c in zm.CONFIGS.items():
        mc = config_from_json(c)
        assert zagolix_json(mc) == c and mc.arch == "zagolix" and architecture(mc).name == "zagolix" and mc.tie_embeddings
        assert mc.is_recurrent == (name != "wide")
        assert mc.n_params() == sum(int(np.prod(x.shape)) for x in zm.weights(c).values())
    mc = zagolix_config(zm.CONFIGS["mixed"])
    assert mc.active_params() == mc.n_params() - 3 * 160 * ((15 - 2) * 40 + (8 - 3) * 72 + (12 - 1) * 36)
    # two maps of keys and one of values; one latent row for three layers; nothing for the memory
    assert mc.kv_bytes_per_token() == 2 * (2 * (64 + 48) + 3 * (80 + 96) + 72 + 12)
    bad = [("layers", 0, "type", "ssd"), ("layers", 2, "mixer", "kv_heads", 3), ("layers", 0, "mlp", "router", "top", 7),
           ("layers", 0, "mlp", "router", "groups", {"count": 4, "keep": 2}), ("layers", 4, "mlp", "router", "groups", {"count": 3, "keep": 4}),
           ("layers", 2, "mlp", "router", "top", 9), ("layers", 1, "mlp", "kind", "glu"), ("layers", 3, "mixer", "kv_from", 3),
           ("layers", 3, "mixer", "kv_from", 2), ("layers", 5, "mixer", "kv_from", 3), ("layers", 3, "mixer", "kv_rank", 64),
           ("layers", 1, "mixer", "rot", {"base": 1000.0, "dims": 10}), ("layers", 5, "mixer", "rot", {"base": 999.0, "dims": 12})]
    for b in bad:
        with pytest.raises(ConfigError):
            zagolix_config(changed(zm.CONFIGS["mixed"], setting(*b)))


def test_weights_load_from_a_model_folder(tmp_path):
    c = zm.CONFIGS["mixed"]
    w = zm.weights(c, 3)
    assert not any(n.startswith(("l3.mix.dkv", "l5.mix.dkv")) for n in w) and "head" not in w and "l3.norm2" not in w
    hm.write_model(tmp_path / "m", c, w)
    src = open_weights(str(tmp_path / "m"))
    assert src.cfg == zagolix_config(c)
    for n, x in w.items():
        assert np.array_equal(src.f32(n), x), n
    for bad in ("l0.mlp.e3.gate", "l1.mix.uk", "l2.mix.k.b"):
        w2 = dict(w)
        w2[bad] = w2[bad][:-1]
        hm.write_model(tmp_path / "bad", c, w2)
        with pytest.raises(ModelLoadError):
            open_weights(str(tmp_path / "bad"))


def test_synthetic_weights_start_with_open_memories():
    mc = preset("zagolix-tiny")
    src = SyntheticSource(mc, seed=1)
    assert src.f32("l3.mix.f.b").min() >= 3 and np.all(src.f32("l0.mix.lq1") == 0) and np.all(src.f32("l1.ls2") == 1)
    assert np.all(src.f32("l0.mix.q.b") == 0) and {n for n, _ in tensor_names(mc)} == set(src.names())


def test_passes_over_the_contexts_of_prompts():
    """Every prompt's context gets whole pages of rows; passes hold a bounded number of them, longer ones one prompt."""
    from types import SimpleNamespace

    from oxide_tech_llm_engine_b200.engine.engine import LLMEngine
    from oxide_tech_llm_engine_b200.models import hybrid

    rng = np.random.default_rng(3)
    for _ in range(50):
        n = int(rng.integers(1, 9))
        q = rng.integers(1, 400, size=n)
        ctx = q + rng.integers(0, 3, size=n) * rng.integers(0, 40000, size=n)
        start = np.full(n, -1, dtype=np.int32)
        passes = LLMEngine._kv_passes(SimpleNamespace(ctx_lens=ctx, q_lens=q, n_prefill=n), start)
        assert [p[0] for p in passes] + [n] == [0] + [p[1] for p in passes]
        tile = 0
        for s0, s1, t0, t1, rows, pages in passes:
            at = 0
            for i in range(s0, s1):
                assert start[i] == at
                at += (ctx[i] + 15) // 16 * 16
            assert rows == at and (rows <= hybrid.KV_PASS_ROWS or s1 == s0 + 1)
            assert t0 == tile and t1 - t0 == sum((q[s0:s1] + 127) // 128) and pages == max((ctx[s0:s1] + 15) // 16)
            tile = t1


# ---------------------------------------------------------------- the plain implementation is sharp
def test_the_test_models_show_every_mistake():
    """A planted mistake in the plain implementation moves the logits by far more than the tolerances."""
    c = zm.CONFIGS["mixed"]
    w, t = zm.weights(c, 1), toks(150, 300, 5)
    good = oracle.forward(c, w, t).numpy()

    def off(cfg=None, weights=w, **patch):
        with pytest.MonkeyPatch.context() as mp:
            for name, fn in patch.items():
                mp.setattr(oracle, name, fn)
            return hm.error(oracle.forward(changed(c, setting(*cfg)) if cfg else c, weights, t).numpy(), good)

    o = oracle
    mlstm, diff, rotate, latent, temperature, choose, causal = (o.mlstm, o.differential, o.rotate_pairs, o.latent, o.temperature, o.choose, o.causal)

    def other_map_order(q, k, v, s, lam, d, e):
        return diff(q.flip(2), k.flip(2), v, s, lam, d, e)

    def without_max(q, k, v, i, f):            # the denominator's floor is exp(-m): without m it is another one
        return mlstm(q, k, v, i - 3.0, f)

    def state_of_one_chunk(q, k, v, i, f):
        cut = [mlstm(x[:64], y[:64], z[:64], a[:64], b[:64])[0] for x, y, z, a, b in ((q, k, v, i, f),)]
        rest = mlstm(q[64:], k[64:], v[64:], i[64:], f[64:])[0]
        return torch.cat([cut[0], rest]), None

    def flipped_uv(z):
        return {**z, "l1.mix.uk": z["l1.mix.uk"].reshape(5, 24, 72)[::-1].reshape(-1, 72).copy()}

    swap = lambda a, b: {**w, a: w[b], b: w[a]}
    cases = {
        "other map first": off(differential=other_map_order), "no second map": off(map_weight=lambda *a: 0.0 * a[0].sum()),
        "diff": off(("layers", 2, "mixer", "diff", 0.5)), "map weight": off(map_weight=lambda a, b, c_, d, e: e + 0 * a.sum()),
        "keys' maps": off(differential=lambda q, k, v, s, l, d, e: diff(q, k.flip(2), v, s, l, d, e)),
        "temperature": off(temperature=lambda p, a, b: temperature(p + 1, a, b)), "no temperature": off(temperature=lambda p, a, b: 1 + 0 * temperature(p, a, b)),
        "biases": off(weights={n: (0 * x if n.endswith(("q.b", "k.b", "v.b")) else x) for n, x in w.items()}),
        "a key ahead": off(causal=lambda q, k, v, s: causal(q, k.roll(1, 0), v, s)),
        "no rotation": off(rotate_pairs=lambda x, p, b: x), "base": off(("layers", 1, "mixer", "rot", "base", 900.0)),
        "rotation of the halves": off(rotate_pairs=lambda x, p, b: rotate(x[..., torch.randperm(12, generator=torch.Generator().manual_seed(1))], p, b)),
        "keys one further": off(latent=lambda m, z, p, h, pos, e: latent(m, z, p, h, pos + 1, e)),
        "latent not normed": off(latent=lambda m, z, p, h, pos, e: ((h @ z[p + "dkv"].T)[:, :m["kv_rank"]], latent(m, z, p, h, pos, e)[1])),
        "heads of W_uk": off(weights=flipped_uv(w)),
        "no running maximum": off(mlstm=without_max), "state lost": off(mlstm=state_of_one_chunk),
        "gates swapped": off(mlstm=lambda q, k, v, i, f: mlstm(q, k, v, f, -torch.log1p(torch.exp(-i)))),
        "cap": off(("layers", 0, "mixer", "gate_cap", 3.0)), "gate and scores": off(sigmoid=lambda z: 0.5 + 0.5 * z.tanh()),
        "top": off(("layers", 0, "mlp", "router", "top", 1)), "no groups": off(choose=lambda lg, k, g=None: choose(lg, k, None)),
        "keep": off(("layers", 0, "mlp", "router", "groups", "keep", 1)),
        "weights divided": off(choose=lambda lg, k, g=None: (choose(lg, k, g)[0], choose(lg, k, g)[1] / choose(lg, k, g)[1].sum(-1, keepdim=True))),
        "dense act": off(gelu_tanh=o.silu), "expert act": off(silu=o.gelu_tanh),
        "norms swapped": off(weights=swap("l0.norm1", "l0.norm1b")), "layer scales swapped": off(weights=swap("l1.ls1", "l1.ls2")),
        "eps": off(("norm", "eps", 1e-2)), "scale": off(("embedding", "scale", 2.0)), "score scale": off(("layers", 1, "mixer", "scale", 0.2)),
    }
    shared = changed(c, lambda x: None)
    shared["layers"].insert(2, zm.lat(2, 16, 16, 20, 72, 12))       # another latent that later layers could read by mistake
    for i in (4, 6):
        shared["layers"][i]["mixer"]["kv_from"] = 1
    ws = zm.weights(shared, 1)
    a = oracle.forward(shared, ws, t).numpy()
    shared["layers"][4]["mixer"]["kv_from"] = 2
    cases["another layer's latents"] = hm.error(oracle.forward(shared, ws, t).numpy(), a)
    assert all(v > 0.02 for v in cases.values()), {k: v for k, v in cases.items() if not v > 0.02}


def test_choice_by_groups_in_the_plain_implementation():
    """The best single expert in a poor group is not chosen; the second largest score of a group counts, the third does not."""
    z = torch.tensor([[3.0, -9, -9, 1.0, 0.9, -9, 0.8, 0.8, 0.8]], dtype=torch.float64)
    ids, s = oracle.choose(z, 2, {"count": 3, "keep": 1})
    assert ids.tolist() == [[3, 4]] and torch.allclose(s, torch.sigmoid(z[:, 3:5]))
    assert oracle.choose(z, 2)[0].tolist() == [[0, 3]] and oracle.choose(z, 3, {"count": 3, "keep": 2})[0].tolist() == [[3, 4, 6]]


# ---------------------------------------------------------------- engine on the CPU backend
@pytest.mark.parametrize("name", list(zm.CONFIGS))
def test_cpu_engine_equals_the_plain_implementation(name):
    c = zm.CONFIGS[name]
    w = zm.weights(c, 2)
    eng = hm.engine(c, w, backend="cpu", live=2, blocks=24)
    seqs = [toks(n, c["vocab"], n) for n in (1, 45, 90, 2, 33)]
    want = [oracle.forward(c, w, t).numpy() for t in seqs]
    for t, x in zip(seqs, want):
        assert hm.error(hm.feed_all(eng, 0, t, []), x) < 1e-4
        assert hm.error(hm.feed_all(eng, 0, t, [2, 3, 1, 1, 17, 2]), x) < 1e-4
    for got, x in zip(hm.interleaved(eng, seqs, 11), want):
        assert hm.error(got, x) < 1e-4
    assert eng.sched.num_free_blocks() == 24 and (name == "wide" or eng.sched.num_free_slots() == 2)


def test_cpu_generation_through_the_scheduler_is_greedy_decoding():
    c = zm.CONFIGS["mixed"]
    w = zm.weights(c, 4)
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


def test_prefix_cache_shares_latents_of_models_without_state():
    c = zm.CONFIGS["wide"]
    w = zm.weights(c, 4)
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

    c = zm.model(64, 256, [zm.dense(zm.att(2, 1, 16, 32), 48), zm.moe(zm.lat(2, 16, 24, 24, 32, 8), 6, 2, 40, (2, 1)), zm.mem(2, 16, 32)])
    hm.write_model(tmp_path / "m", c, zm.weights(c, 1))
    for m in (str(tmp_path / "m"), "zagolix-tiny"):
        assert cli.main(["verify", "-m", m, "-b", "cpu", "--greedy", "-c", "256", "--max-slots", "2"]) == 0
        assert len(json.loads(capsys.readouterr().out.strip().splitlines()[-1])["tokens"]) == 16


def test_refused_options():
    c = zm.CONFIGS["ones"]
    for kw in (dict(h2o_pruning=True), dict(context_shift=True), dict(comm="nccl")):
        with pytest.raises(ConfigError):
            hm.engine(c, zm.weights(c), backend="cpu", **kw)
