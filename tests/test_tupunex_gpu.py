"""Tupunex on the GPU through the replay program and the engine: every cutting of the work against the plain
implementation, in both number formats, for configurations that differ in every size and option."""
import pytest
import torch

import helpers
import tupunex_helpers as XH

pytestmark = pytest.mark.gpu

BF16_TOP1 = 0.9


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, name in enumerate(XH.CONFIGS):
        d = str(tmp_path_factory.mktemp("tupunex" + name))
        XH.make_model(d, name, seed=50 + i)
        out[name] = (d,) + XH.CONFIGS[name]
    return out


# lengths around the windows' edges (9 and 30; 64 and none; 5 and 21; 17) and the pages', and the sizes from which a step's rows
# are prepared several tokens at a time; more requests than state slots, so that slots come back
LENGTHS = {"U": (1, 2, 9, 10, 31, 43, 90, 131, 64), "V": (3, 64, 65, 33, 160, 48), "W": (5, 6, 21, 22, 64, 130, 200, 8), "X": (17, 18, 1, 150, 40)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(XH.CONFIGS))
def test_every_cutting_matches_plain(name, dtype, models, tmp_path):
    d, cfg, page = models[name]
    seqs = helpers.random_tokens(cfg["vocab"], LENGTHS[name], seed=3)
    ref = XH.plain_logits(d, cfg, seqs)
    families = {
        "w": helpers.trace_whole(seqs, tag="w"),
        "t": helpers.trace_tail(seqs, tail=48, tag="t"),           # decoding passes windows' edges
        "c": helpers.trace_chunks(seqs, tag="c"),                  # portions of 1 to 11 tokens
        "m": helpers.trace_mixed(seqs, tag="m"),
        "n": helpers.trace_mixed(seqs, sizes=(140, 2, 37, 1, 64), tag="n", seed=1),  # long portions beside single tokens
    }
    steps = [s for f in families.values() for s in f]
    longest = sorted((len(v) for v in seqs.values()), reverse=True)[:4]
    max_tokens = sum(-(-n // 64) * 64 for n in longest)             # pages and slots are used again
    steps, out = helpers.run_trace(d, dtype, steps, str(tmp_path), max_tokens, page)
    tol = helpers.FP32_TOL if dtype == "float32" else helpers.BF16_TOL
    # a place that amplifies every rounding is judged by what rounding does to the plain implementation there
    rounding = XH.rounding_errors(d, cfg, seqs, ref, getattr(torch, dtype))
    for tag in families:
        sub = [s for s in steps if s["entries"][0]["id"].startswith(tag)]
        worst, where, agree, clear = helpers.compare_trace(sub, out, cfg["vocab"], ref, rounding=rounding, unit=tol)
        assert worst <= tol, f"family {tag!r}: error {worst:.3g} of the logit scale at (step, request, position) {where}"
        if dtype == "float32":
            assert agree == 1.0, f"family {tag!r}: greedy tokens differ from the plain implementation"
        else:
            assert agree >= BF16_TOP1 and clear == 1.0, f"family {tag!r}: top-1 agreement {agree:.3f} ({clear:.3f} where clear)"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_one_token_at_a_time(dtype, models, tmp_path):
    """A short prompt, then hundreds of single-token steps through the captured decode graph: windows pass over decoded tokens,
    their pages come back, the convolution's rings are carried through every step of every pass."""
    d, cfg, page = models["U"]
    seq = helpers.random_tokens(cfg["vocab"], (330,), seed=11)
    ref = XH.plain_logits(d, cfg, seq)
    steps, out = helpers.run_trace(d, dtype, helpers.trace_tail(seq, tail=322), str(tmp_path), 384, page)
    tol = helpers.FP32_TOL if dtype == "float32" else helpers.BF16_TOL
    worst, where, agree, clear = helpers.compare_trace(steps, out, cfg["vocab"], ref, unit=tol,
                                                       rounding=XH.rounding_errors(d, cfg, seq, ref, getattr(torch, dtype)))
    assert worst <= tol, (worst, where)
    assert agree == 1.0 if dtype == "float32" else agree > 0.9


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_in_one_step_and_in_two(dtype, models, tmp_path):
    """Seven hundred tokens at once (rows sixteen tokens a block, attention over dozens of pages), and the same cut at a place
    that is no edge of anything."""
    d, cfg, page = models["V"]
    seq = helpers.random_tokens(cfg["vocab"], (700,), seed=5)
    ref = XH.plain_logits(d, cfg, seq)
    v = seq["r0"]
    steps = helpers.trace_whole(seq, tag="w") + [
        {"entries": [{"id": "cr0", "tokens": v[:389], "want": list(range(0, 389, 7))}], "end": []},
        {"entries": [{"id": "cr0", "tokens": v[389:], "want": list(range(311))}], "end": ["cr0"]}]
    steps, out = helpers.run_trace(d, dtype, steps, str(tmp_path), 1536, page)
    tol = helpers.FP32_TOL if dtype == "float32" else helpers.BF16_TOL
    worst, where, agree, _ = helpers.compare_trace(steps, out, cfg["vocab"], ref, unit=tol,
                                                   rounding=XH.rounding_errors(d, cfg, seq, ref, getattr(torch, dtype)))
    assert worst <= tol and agree > (0.999 if dtype == "float32" else 0.9), (worst, where, agree)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_generation_through_the_engine(dtype, models):
    """Greedy tokens through the entry point and the scheduler, with few pages and a small token budget (prompts in
    portions, preemption and recomputation, slots used again), against the plain loop."""
    from atoma_infer_b200.engine import Engine
    from atoma_infer_b200.sampling import SamplingParams
    import plain_tupunex as PX

    d, cfg, page = models["W"]
    prompts = list(helpers.random_tokens(cfg["vocab"], (3, 70, 9, 130, 21), seed=8).values())
    eng = Engine(d, dtype=dtype, block_size=page, num_gpu_blocks_override=40, max_num_sequences=3, max_num_batched_tokens=48)
    outs = eng.generate(prompts, SamplingParams(do_sample=False, max_new_tokens=12, ignore_eos_token=True))
    eng.lm.rt.ops.check_status()
    assert eng.lm.manager.audit() == "" and eng.lm.manager.num_requests() == 0
    w = helpers.read_weights(d)
    for p, o in zip(prompts, outs):
        got = o.token_ids
        if dtype == "float32":
            assert got == XH.plain_greedy(d, cfg, p, 12)
            continue
        logits = PX.forward(cfg, w, list(p) + list(got))  # each token judged on the engine's own history
        for i, tok in enumerate(got):
            row = logits[len(p) - 1 + i]
            lead = float(row.max() - row[tok]) / float(row.abs().max())
            assert lead <= 2 * helpers.BF16_TOL, (i, tok, lead)


def test_the_command_line_serves_the_design(tmp_path):
    """``random-model`` writes a Tupunex folder from its configuration, ``generate`` decodes greedily from it; both as
    child processes, the tokens against the plain loop (float32)."""
    import json
    import os
    import subprocess
    import sys

    cli = os.path.join(helpers.ROOT, "bin", "atoma-infer")
    cfg, page = XH.CONFIGS["V"]
    (tmp_path / "config_in.json").write_text(json.dumps(cfg))
    out = tmp_path / "model"

    def run(args):
        p = subprocess.run([sys.executable, cli, *args], capture_output=True, text=True, timeout=900)
        assert p.returncode == 0, f"atoma-infer {' '.join(args)} failed ({p.returncode}):\n{p.stdout[-2000:]}\n{p.stderr[-4000:]}"
        return p

    run(["random-model", "--config", str(tmp_path / "config_in.json"), "--seed", "7", "--out", str(out), "--std", "0.05",
         "--norm-jitter", "0.1"])
    prompts = [[3, 14, 15, 92, 65, 35, 89, 79], list(range(40, 95))]
    args = ["generate", "--model", str(out), "--dtype", "f32", "--block-size", str(page), "--num-gpu-blocks-override", "16",
            "--max-num-batched-tokens", "24", "--max-num-sequences", "2", "--no-do-sample", "--max-new-tokens", "8",
            "--ignore-eos-token"]
    for p in prompts:
        args += ["--prompt-ids", ",".join(map(str, p))]
    recs = [json.loads(line) for line in run(args).stdout.splitlines() if line.startswith("{")]
    assert [r["token_ids"] for r in recs] == [XH.plain_greedy(str(out), cfg, p, 8) for p in prompts]
