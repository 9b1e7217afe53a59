"""Kavotar through the engine's host side without a GPU: configuration, weights by name, the block with norms on the results
and its mixers' shares of a request's state, pages and slots used again, the scheduler.  The kernels are the torch stand-ins
of host_ops.py; what the CUDA kernels compute is tested on the GPU."""
import io
import json

import pytest
import torch

import helpers
import kavotar_helpers as VH
from host_ops import HostOps

SEEDS = {"U": 40, "V": 42, "W": 42}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name in VH.CONFIGS:
        d = str(tmp_path_factory.mktemp("kavotar" + name))
        VH.make_model(d, name, seed=SEEDS[name])
        out[name] = (d,) + VH.CONFIGS[name]
    return out


def _replay(d, steps, out_dir, max_tokens, page):
    from atoma_infer_b200.engine.trace import replay

    steps = helpers.number(steps)
    text = "\n".join(json.dumps(s) for s in steps) + "\n"
    replay(d, "float32", out_dir, max_tokens, stream=io.StringIO(text), out=io.StringIO(), page_size=page, device="cpu",
           ops=HostOps())
    return steps


@pytest.mark.parametrize("name", list(VH.CONFIGS))
def test_every_cutting_matches_plain(name, models, tmp_path):
    d, cfg, page = models[name]
    seqs = helpers.random_tokens(cfg["vocab"], (1, 2, 9, 30, 47), seed=5)
    ref = VH.plain_logits(d, cfg, seqs)
    steps = (helpers.trace_whole(seqs) + helpers.trace_tail(seqs, tail=12) + helpers.trace_chunks(seqs, sizes=(5, 2, 7, 3, 2, 11, 1, 4))
             + helpers.trace_mixed(seqs, sizes=(6, 2, 9, 3, 5)))
    steps = _replay(d, steps, str(tmp_path), 192, page)  # four live requests at most, 64 tokens each: pages come back
    worst, where, agree, _ = helpers.compare_trace(steps, str(tmp_path), cfg["vocab"], ref, unit=helpers.FP32_TOL,
                                                  rounding=VH.rounding_errors(d, cfg, seqs, ref, torch.float32))
    assert worst <= helpers.FP32_TOL, (worst, where)
    assert agree == 1.0


def test_config_is_read_key_by_key():
    from atoma_infer_b200.config import ConfigError
    from atoma_infer_b200.config.kavotar_config import KavotarConfig, MemorySizes, SideBySideSizes

    cfg = VH.CONFIGS["U"][0]
    c = KavotarConfig.from_dict(cfg)
    assert (c.width, c.vocab, c.eps, c.logit_softcap) == (96, 131, 1e-5, 12.0)
    mem, both, mem2 = (ly.mixer for ly in c.layers)
    assert mem == MemorySizes(heads=3, dim=16, vdim=40, gate_cap=6.0) and mem2.gate_cap == 2.5
    assert isinstance(both, SideBySideSizes)
    a = both.left
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk, a.rot_dims, a.rot_base) == (6, 3, 32, 16, 0.3, 12, 16, 200.0)
    assert (both.right.heads, both.right.dim) == (3, 24)
    f = c.layers[0].mlp
    assert (f.ff, f.experts, f.top, f.groups) == (40, 8, 2, (4, 2)) and c.layers[2].mlp is None
    # what an entry does not mention is off
    v = KavotarConfig.from_dict(VH.CONFIGS["V"][0])
    assert (v.layers[0].mixer.left.chunk, v.layers[2].mixer.left.rot_dims, v.layers[0].mlp.groups, v.logit_softcap) == (None, 0, None, None)

    def broken(edit, match):
        bad = json.loads(json.dumps(cfg))
        edit(bad)
        with pytest.raises(ConfigError, match=match):
            KavotarConfig.from_dict(bad)

    broken(lambda b: b["layers"][0].update(type="slstm"), "slstm")
    broken(lambda b: b["layers"][0]["mixer"].pop("gate_cap"), "gate_cap")
    broken(lambda b: b["layers"][0]["mixer"].update(gate_cap=0.0), "gate_cap")
    broken(lambda b: b["layers"][1]["mixer"]["left"].update(kv_heads=4), "kv_heads")
    broken(lambda b: b["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "rot.dims")
    broken(lambda b: b["layers"][1]["mixer"]["left"]["mask"].update(size=0), "mask.size")
    broken(lambda b: b["layers"][1]["mixer"].pop("right"), "right")
    broken(lambda b: b["layers"][0]["mlp"].update(kind="dense"), "dense")
    broken(lambda b: b["layers"][0]["mlp"]["router"].update(top=9), "top")
    broken(lambda b: b["layers"][0]["mlp"]["router"]["groups"].update(count=3), "groups")
    broken(lambda b: b["layers"][0]["mlp"]["router"].update(top=5), "groups")


def test_the_spec_puts_each_mechanism_where_the_configuration_says(models):
    from atoma_infer_b200.engine.runtime import load_model

    d, cfg, page = models["U"]
    lm = load_model(d, dtype="float32", device="cpu", ops=HostOps(), num_pages=16, page_size=page, max_seqs=2)
    blocks = lm.model.blocks
    assert [type(b).__name__ for b in blocks] == ["ResultNormBlock"] * 3
    assert [type(b.mixer).__name__ for b in blocks] == ["MatrixMemory", "SideBySide", "MatrixMemory"]
    both = blocks[1].mixer
    assert both.scales == (0.5, 0.5) and both.out_norm is not None and type(both.right).__name__ == "TokenMixing"
    assert (both.left.talk, both.left.head_scale, both.left.head_norm_weight, both.left.chunk) == (True, True, True, 12)
    assert both.right.w1.shape == (16, 96)                        # the decay map's width is the checkpoint's
    assert blocks[2].feed_forward is None and blocks[0].feed_forward.groups == (4, 2) and blocks[0].feed_forward.sigmoid
    assert type(blocks[0].norm1).__name__ == "LayerNorm" and lm.model.head.softcap == 12.0
    # the state of a request: matrices, normalizers and maxima, each on 16 bytes; a kept row and matrices
    assert blocks[0].state_bytes() == (3 * 16 * 40 + 3 * 16 + 4) * 4 and blocks[2].state_bytes() == (48 * 24 + 48 + 4) * 4
    assert blocks[1].state_bytes() == (96 + 3 * 24 * 24) * 4
    assert both.cache_need().chunk == 12 and blocks[0].mixer.cache_need() is None
    # side by side in a model whose sizes are no multiple of four: the shares still start on 16 bytes
    dw, _, pw = models["W"]
    lw = load_model(dw, dtype="float32", device="cpu", ops=HostOps(), num_pages=16, page_size=pw, max_seqs=2)
    mem = lw.model.blocks[1].mixer
    S, n, m = mem.states(torch.zeros((3, mem.state_bytes()), dtype=torch.uint8))
    assert S.shape == (3, 2, 10, 14) and n.shape == (3, 2, 10) and m.shape == (3, 2)
    assert all(t.storage_offset() % 4 == 0 for t in (S, n, m))


def test_a_missing_tensor_is_named(models, tmp_path):
    from atoma_infer_b200.engine.runtime import load_model
    from atoma_infer_b200.weights.loader import WeightError
    from atoma_infer_b200.weights.safetensors_io import write_safetensors

    d, cfg, page = models["U"]
    w = {k: v.to(torch.bfloat16) for k, v in helpers.read_weights(d).items()}
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    for name in ("l0.mix.f.b", "l1.mix.left.talk", "l1.mix.left.temp", "l1.mix.right.mu.w", "l1.mix.right.out", "l0.mlp.correction", "head",
                 "l1.mix.right.u"):
        gone = dict(w)
        del gone[name]
        write_safetensors(str(tmp_path / "model.safetensors"), gone, {})
        with pytest.raises(WeightError, match=name):
            load_model(str(tmp_path), dtype="float32", device="cpu", ops=HostOps(), num_pages=8, page_size=page, max_seqs=2)
    # the two factors of the decay map must agree on its width, whatever it is
    for wide, ok in ((5, True), (7, False)):
        other = dict(w, **{"l1.mix.right.w1": torch.zeros(5, 96, dtype=torch.bfloat16), "l1.mix.right.w2": torch.zeros(72, wide, dtype=torch.bfloat16)})
        write_safetensors(str(tmp_path / "model.safetensors"), other, {})
        if ok:
            load_model(str(tmp_path), dtype="float32", device="cpu", ops=HostOps(), num_pages=8, page_size=page, max_seqs=2)
        else:
            with pytest.raises(WeightError, match="right.w2"):
                load_model(str(tmp_path), dtype="float32", device="cpu", ops=HostOps(), num_pages=8, page_size=page, max_seqs=2)


def test_normed_terms_are_made_first_where_another_block_takes_the_sum():
    """A pending sum whose terms carry norms of their own, handed to a consumer that knows none."""
    from atoma_infer_b200.parts.base import PendingSum, join_terms, without_norms
    import kernel_utils as K
    from atoma_infer_b200.parts.base import Runtime
    import plain_kavotar as PV

    rt = Runtime(torch.device("cpu"), torch.float32, HostOps())
    ctx, _ = K.make_context(rt, [(0, 4)], 16, [[1]])
    a, b, w = torch.randn(4, 6), torch.randn(4, 6), torch.rand(6)
    pend = PendingSum((a, b), 1.0, factors=(0.5, 0.25), norms=((w, 1e-5), None))
    out = without_norms(rt.ops, pend, ctx)
    assert out.norms is None and torch.allclose(out.terms[0], PV.rms(a, 1e-5) * w, atol=1e-6) and out.terms[1] is b and out.factors == (0.5, 0.25)
    with pytest.raises(ValueError):
        join_terms((pend,))


def test_greedy_generation_through_the_scheduler(models):
    """Few pages and a small token budget: prompts are cut, requests preempted and recomputed, slots used again."""
    from atoma_infer_b200.engine import Engine
    from atoma_infer_b200.sampling import SamplingParams

    d, cfg, page = models["V"]
    prompts = list(helpers.random_tokens(cfg["vocab"], (3, 26, 9, 17, 5), seed=8).values())
    want = [VH.plain_greedy(d, cfg, p, 10) for p in prompts]
    eng = Engine(d, dtype="float32", block_size=page, cuda_graphs=False, ops=HostOps(), num_gpu_blocks_override=6,
                 max_num_sequences=3, max_num_batched_tokens=11)
    outs = eng.generate(prompts, SamplingParams(do_sample=False, max_new_tokens=10, ignore_eos_token=True))
    assert [o.token_ids for o in outs] == want
    assert eng.lm.manager.audit() == "" and eng.lm.manager.num_requests() == 0
