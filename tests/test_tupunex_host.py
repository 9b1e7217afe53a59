"""Tupunex through the engine's host side without a GPU: configuration, weights by name, blocks on several streams and what they
leave pending, layers that run several times with a cache and a state of their own, the convolution's ring by slot, windows
whose pages go back, the scheduler.  The kernels are the torch stand-ins of host_ops.py; what the CUDA kernels compute is
tested on the GPU."""
import io
import json

import pytest
import torch

import helpers
import tupunex_helpers as XH
from host_ops import HostOps


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, name in enumerate(XH.CONFIGS):
        d = str(tmp_path_factory.mktemp("tupunex" + name))
        XH.make_model(d, name, seed=50 + i)
        out[name] = (d,) + XH.CONFIGS[name]
    return out


def _load(d, page, **kw):
    from atoma_infer_b200.engine.runtime import load_model

    return load_model(d, dtype="float32", device="cpu", ops=HostOps(), page_size=page, **{"num_pages": 16, "max_seqs": 2, **kw})


def _replay(d, steps, out_dir, max_tokens, page):
    from atoma_infer_b200.engine.trace import replay

    steps = helpers.number(steps)
    text = "\n".join(json.dumps(s) for s in steps) + "\n"
    replay(d, "float32", out_dir, max_tokens, stream=io.StringIO(text), out=io.StringIO(), page_size=page, device="cpu",
           ops=HostOps())
    return steps


@pytest.mark.parametrize("name", list(XH.CONFIGS))
def test_every_cutting_matches_plain(name, models, tmp_path):
    d, cfg, page = models[name]
    seqs = helpers.random_tokens(cfg["vocab"], (1, 2, 9, 30, 47), seed=5)
    ref = XH.plain_logits(d, cfg, seqs)
    steps = (helpers.trace_whole(seqs) + helpers.trace_tail(seqs, tail=12) + helpers.trace_chunks(seqs, sizes=(5, 2, 7, 3, 2, 11, 1, 4))
             + helpers.trace_mixed(seqs, sizes=(6, 2, 9, 3, 5)))
    steps = _replay(d, steps, str(tmp_path), 192, page)  # four live requests at most, 64 tokens each: pages come back
    worst, where, agree, _ = helpers.compare_trace(steps, str(tmp_path), cfg["vocab"], ref, unit=helpers.FP32_TOL,
                                                  rounding=XH.rounding_errors(d, cfg, seqs, ref, torch.float32))
    assert worst <= helpers.FP32_TOL, (worst, where)
    assert agree == 1.0


def test_the_streams_after_every_layer_run(models):
    """The sum of the streams with what is pending taken in, after every run of the schedule, against the plain
    implementation's: a layer that runs again counts each time."""
    from types import SimpleNamespace

    import plain_tupunex as PX
    from atoma_infer_b200.engine.step import StepEntry
    from atoma_infer_b200.parts.base import StreamMix, apply_pending

    d, cfg, page = models["U"]
    toks = helpers.random_tokens(cfg["vocab"], (19,), seed=2)["r0"]
    want = []
    PX.forward(cfg, helpers.read_weights(d), toks, layers_out=want)
    lm = _load(d, page)
    got, seen, run = [], [], lm.model.forward
    lm.model.forward = lambda ctx, *a: seen.append(ctx) or run(ctx, *a)

    def watch(i, resid, delta):
        assert isinstance(delta, StreamMix) and resid.shape == (len(toks), 3 * 96)
        x = resid.clone()
        apply_pending(lm.rt.ops, x, delta, SimpleNamespace(meta=seen[0].meta, T=len(toks)))
        got.append(x.view(len(toks), 3, 96).sum(1))

    lm.model.watch = watch
    lm.step.run([StepEntry(0, toks, [len(toks) - 1])])
    assert len(got) == len(want) == 2 * 2 + 1
    for a, b in zip(got, want):
        assert float((a.double() - b).abs().max()) < 1e-4 * float(b.abs().max())


def test_config_is_read_key_by_key():
    from atoma_infer_b200.config import ConfigError
    from atoma_infer_b200.config.tupunex_config import DifferentialAttentionSizes, SharedLatentSizes, TupunexConfig

    cfg = XH.CONFIGS["U"][0]
    c = TupunexConfig.from_dict(cfg)
    assert (c.width, c.vocab, c.eps, c.embedding_scale, c.streams) == (96, 131, 1e-5, 3.0, 3)
    assert (c.loop.start, c.loop.stop, c.loop.times) == (0, 2, 2)
    assert c.layers[0].mixer == DifferentialAttentionSizes(heads=4, kv_heads=2, dim=16, vdim=32, scale=0.5, diff=0.35, conv=4, softcap=3.0, window=9)
    assert c.layers[1].mixer == SharedLatentSizes(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, scale=0.4, rot_dims=8, rot_base=1e4)
    assert c.layers[0].mlp.ff == 160 and c.layers[2].mlp is None
    v = TupunexConfig.from_dict(XH.CONFIGS["V"][0])   # what an entry does not mention is off
    assert (v.layers[2].mixer.window, v.layers[2].mixer.softcap, v.layers[2].mixer.conv) == (None, None, 0)
    assert TupunexConfig.from_dict(XH.CONFIGS["X"][0]).loop is None
    for path, value, word in ((("layers", 0, "type"), "mlstm", "mlstm"), (("layers", 0, "mlp", "kind"), "moe", "moe"),
                              (("layers", 0, "mixer", "diff"), None, "diff"), (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
                              (("layers", 0, "mixer", "mask", "size"), 0, "mask.size"), (("layers", 0, "mixer", "conv"), -1, "conv"),
                              (("layers", 1, "mixer", "kv_rank"), None, "kv_rank"), (("layers", 1, "mixer", "rot", "dims"), 10, "rot.dims"),
                              (("loop", "stop"), 7, "loop"), (("streams",), 0, "streams"), (("norm", "eps"), None, "eps")):
        bad = json.loads(json.dumps(cfg))
        at = bad
        for key in path[:-1]:
            at = at[key]
        if value is None:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            TupunexConfig.from_dict(bad)


def test_the_spec_puts_each_mechanism_where_the_configuration_says(models):
    d, cfg, page = models["U"]
    m = _load(d, page).model
    assert [r.layer for r in m.runs] == [0, 1, 0, 1, 2] and m.run_owner == list(range(5))   # no run reads another's cache
    assert [type(b).__name__ for b in m.blocks] == ["HyperBlock"] * 3 and {b.streams for b in m.blocks} == {3}
    assert [type(b.mixer).__name__ for b in m.blocks] == ["Attention", "LatentAttention", "Attention"]
    a = m.blocks[0].mixer
    assert (a.maps, a.padded_dim, a.taps, a.softcap, a.window, a.head_gate) == (2, 32, 4, 3.0, 9, True)
    assert a.state_bytes() == 3 * (2 * 4 * 16 + 2 * 2 * 16 + 2 * 32) * 4 and a.ring(torch.zeros(5, a.state_bytes(), dtype=torch.uint8)).shape == (5, 3, 256)
    assert a.w_qkv.shape[0] % 8 == 0 and a.w_o.shape == (96, 4 * 32)
    assert m.blocks[1].mixer.halves and m.blocks[1].mixer.head_gate and m.blocks[1].mixer.w_uq is None
    assert m.blocks[2].feed_forward is None and m.blocks[2].norm2 is None and m.embedding.copies == 3
    # windows of 9 and of 30 over heads of another size, and all keys of the latents: three pools; every pass a layer of its own
    assert [(g.need.window, g.layers) for g in m.groups] == [(9, [0, 2]), (None, [1, 3]), (30, [4])]
    assert [b > 0 for b in m.state_bytes] == [True, False, True, False, True]


def test_streams_of_model_and_blocks_must_agree():
    from dataclasses import replace

    from atoma_infer_b200.config.tupunex_config import TupunexConfig
    from atoma_infer_b200.models.tupunex import tupunex_spec
    from atoma_infer_b200.parts.model import DecoderModel, LayerRun, StreamAdd

    spec = tupunex_spec(TupunexConfig.from_dict(XH.CONFIGS["V"][0]))
    with pytest.raises(ValueError, match="streams"):
        DecoderModel(replace(spec, streams=3))
    with pytest.raises(ValueError, match="streams"):
        DecoderModel(replace(spec, streams=0))
    with pytest.raises(ValueError, match="plain stream"):
        DecoderModel(replace(spec, schedule=[LayerRun(0), LayerRun(1, before=StreamAdd(embedding=True))]))


def test_what_differential_attention_does_not_go_with():
    from atoma_infer_b200.parts.attention import Attention

    base = {"hidden": 32, "num_heads": 4, "num_kv_heads": 2, "head_dim": 8, "scale": 1.0, "differential": {"diff": 0.2, "eps": 1e-5}}
    Attention(base, "a")
    for extra in ({"qk_norm": {"eps": 1e-5}}, {"sink": True}, {"gate": True}, {"talk": True}, {"position": {"kind": "rope", "head_dim": 8}},
                  {"distance_bias": True}, {"window": 4, "keep_first": 1}):
        with pytest.raises(ValueError):
            Attention(dict(base, **extra), "a")
    with pytest.raises(ValueError, match="convolution"):
        Attention(dict({k: v for k, v in base.items() if k != "differential"}, conv=3, bias=True), "a")


def test_a_missing_tensor_is_named(models, tmp_path):
    from atoma_infer_b200.weights.loader import WeightError
    from atoma_infer_b200.weights.safetensors_io import write_safetensors

    d, cfg, page = models["U"]
    w = {k: v.to(torch.bfloat16) for k, v in helpers.read_weights(d).items()}
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    for name in ("l0.hc1.mix", "l1.hc2.in", "l2.hc1.out", "l0.ls2", "l0.mix.q.conv", "l2.mix.v.b", "l0.mix.lk2", "l1.mix.q", "l1.mix.g", "head"):
        gone = dict(w)
        del gone[name]
        write_safetensors(str(tmp_path / "model.safetensors"), gone, {})
        with pytest.raises(WeightError, match=name.replace(".", r"\.")):
            _load(str(tmp_path), page)
    # what surrounds a feed-forward may be there in a layer without one; anything else nobody asked for is refused
    extra = dict(w, **{"l2.norm2": torch.ones(96, dtype=torch.bfloat16), "l2.hc2.mix": torch.eye(3, dtype=torch.bfloat16)})
    write_safetensors(str(tmp_path / "model.safetensors"), extra, {})
    _load(str(tmp_path), page)
    write_safetensors(str(tmp_path / "model.safetensors"), dict(w, **{"l1.mix.dq": torch.ones(4, 96, dtype=torch.bfloat16)}), {})
    with pytest.raises(WeightError, match="l1.mix.dq"):
        _load(str(tmp_path), page)


def test_random_weights_keep_the_streams_apart_from_nothing(tmp_path):
    """Random-weights mode draws mixing matrices around the identity and shares around one, so that a drawn model carries its
    streams through."""
    from atoma_infer_b200.weights import write_random_model

    cfg, page = XH.CONFIGS["V"]
    write_random_model(str(tmp_path), cfg, 3)
    w = helpers.read_weights(str(tmp_path))
    assert torch.equal(w["l0.hc1.mix"], torch.eye(2)) and torch.equal(w["l1.hc2.out"], torch.ones(2)) and torch.equal(w["l2.ls1"], torch.ones(128))


def test_greedy_generation_through_the_scheduler(models):
    """Few pages and a small token budget: prompts are cut, requests preempted and recomputed, slots used again."""
    from atoma_infer_b200.engine import Engine
    from atoma_infer_b200.sampling import SamplingParams

    for name, blocks in (("V", 6), ("U", 22)):
        d, cfg, page = models[name]
        prompts = list(helpers.random_tokens(cfg["vocab"], (3, 26, 9, 17, 5), seed=8).values())
        want = [XH.plain_greedy(d, cfg, p, 10) for p in prompts]
        eng = Engine(d, dtype="float32", block_size=page, cuda_graphs=False, ops=HostOps(), num_gpu_blocks_override=blocks,
                     max_num_sequences=3, max_num_batched_tokens=11)
        outs = eng.generate(prompts, SamplingParams(do_sample=False, max_new_tokens=10, ignore_eos_token=True))
        assert [o.token_ids for o in outs] == want
        assert eng.lm.manager.audit() == "" and eng.lm.manager.num_requests() == 0
