"""The plain Kavotar implementation, mechanism by mechanism, against what each must do."""
import math

import pytest
import torch

import plain_kavotar as PV

F = torch.float64


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F)


def test_layer_norm_takes_the_mean_off_and_has_eps_inside_the_root():
    x, w = torch.tensor([[1.0, 3.0, 5.0, 7.0]], dtype=F), torch.tensor([1.0, 2.0, 1.0, 0.5], dtype=F)
    want = torch.tensor([[-3.0, -1.0, 1.0, 3.0]], dtype=F) / math.sqrt(5.0 + 0.25) * w
    assert torch.allclose(PV.layer_norm(x, w, 0.25), want)
    assert torch.allclose(PV.layer_norm(x + 100.0, w, 0.25), want)


def test_rotation_pairs_the_halves_and_leaves_the_tail():
    x = rnd(9, 2, 10)
    y = PV.rotate_halves(x, 6, 100.0)
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.allclose(y[0], x[0])
    p, i = 7, 2
    a = p * 100.0 ** (-2.0 * i / 6)
    assert torch.allclose(y[p, 1, i], x[p, 1, i] * math.cos(a) - x[p, 1, i + 3] * math.sin(a))
    assert torch.allclose(y[p, 1, i + 3], x[p, 1, i + 3] * math.cos(a) + x[p, 1, i] * math.sin(a))
    q, k = rnd(1, 1, 6, seed=1).expand(9, 1, 6), rnd(1, 1, 6, seed=2).expand(9, 1, 6)
    qr, kr = PV.rotate_halves(q, 6, 100.0), PV.rotate_halves(k, 6, 100.0)  # a product depends on the distance alone
    assert torch.allclose((qr[8, 0] * kr[5, 0]).sum(), (qr[3, 0] * kr[0, 0]).sum())


def test_chunks_are_counted_from_position_zero():
    see = PV.visible(10, 4)
    assert see[3].nonzero().flatten().tolist() == [0, 1, 2, 3] and see[4].nonzero().flatten().tolist() == [4]
    assert see[9].nonzero().flatten().tolist() == [8, 9] and PV.visible(10)[9].all()


def test_weights_are_mixed_after_the_softmax_and_weigh_the_heads_own_values():
    q, k, v, talk = rnd(5, 4, 3), rnd(5, 2, 3, seed=1), rnd(5, 2, 6, seed=2), rnd(4, 4, seed=3)
    p = PV.head_weights(q, k, 0.5, torch.tensor([1.0, 2.0, 0.0, -1.0], dtype=F), PV.visible(5))
    assert torch.allclose(p.sum(-1), torch.ones(4, 5, dtype=F)) and torch.allclose(p[2, 4], torch.full((5,), 0.2, dtype=F))
    s = (q[4, 1] @ k[:, 0].T) * 0.5 * 2.0   # head 1 of key head 0, its temperature
    assert torch.allclose(p[1, 4], torch.softmax(s, 0))
    m = PV.mix_heads(p, talk)
    assert torch.allclose(m[3, 4], sum(talk[3, g] * p[g, 4] for g in range(4)))
    assert torch.allclose(m.sum(-1), talk.sum(1)[:, None].expand(4, 5))   # (they need not sum to one any more)
    o = PV.weighted_values(m, v)
    assert torch.allclose(o[4, 1], m[1, 4] @ v[:, 0]) and torch.allclose(o[4, 2], m[2, 4] @ v[:, 1])
    assert torch.allclose(PV.mix_heads(p, torch.eye(4)), p)


def test_rows_move_toward_the_row_before():
    x, mu = rnd(4, 3), torch.tensor([0.0, 1.0, 0.25], dtype=F)
    y = PV.moved_toward_previous(x, mu)
    assert torch.allclose(y[:, 0], x[:, 0]) and torch.allclose(y[1:, 1], x[:-1, 1]) and y[0, 1] == 0
    assert torch.allclose(y[2, 2], 0.75 * x[2, 2] + 0.25 * x[1, 2])


def test_bonus_state_against_its_unrolled_sum():
    T, H, d, dv = 6, 2, 3, 4
    r, k, v, decay, u = rnd(T, H, d), rnd(T, H, d, seed=1), rnd(T, H, dv, seed=2), torch.rand(T, H, d, dtype=F), rnd(H, d, seed=3)
    o = PV.bonus_state(r, k, v, decay, u)
    for t in range(T):
        for h in range(H):
            want = (u[h] * k[t, h] * r[t, h]).sum() * v[t, h]   # the current token enters through the bonus alone
            for s in range(t):
                a = torch.ones(d, dtype=F)
                for z in range(s + 1, t):                       # (its own step's decay comes before it, the last one's after the read)
                    a = a * decay[z, h]
                want = want + (a * k[s, h] * r[t, h]).sum() * v[s, h]
            assert torch.allclose(o[t, h], want)


def test_memory_does_not_depend_on_the_running_maximum_but_for_its_floor():
    T, d, dv = 7, 3, 4
    q, k, v = rnd(T, 1, d), rnd(T, 1, d, seed=1), rnd(T, 1, dv, seed=2)
    i, f = rnd(T, 1, seed=3) * 3, PV.log_sigmoid(rnd(T, 1, seed=4) * 2)
    o = PV.matrix_memory(q, k, v, i, f)
    m = 0.0
    for t in range(T):
        m = max(float(f[t] + m), float(i[t]))
        S, n = torch.zeros(d, dv, dtype=F), torch.zeros(d, dtype=F)
        for s in range(t + 1):                     # unstabilised: exp of the sum of later forget gates plus the input gate
            wt = torch.exp(i[s, 0] + f[s + 1:t + 1, 0].sum())
            S, n = S + wt * k[s, 0][:, None] * v[s, 0][None, :], n + wt * k[s, 0]
        want = S.T @ q[t, 0] / (max(abs(float(n @ q[t, 0])), 1.0) + 1e-6 * math.exp(m))
        assert torch.allclose(o[t, 0], want), t


def test_memory_starts_with_a_maximum_of_zero():
    one = torch.ones(1, 1, 1, dtype=F)
    o = PV.matrix_memory(one, one, one, torch.full((1, 1), -5.0, dtype=F), torch.full((1, 1), -0.1, dtype=F))
    m = max(-0.1, -5.0)
    assert torch.allclose(o[0, 0, 0], torch.tensor(math.exp(-5.0 - m) / (math.exp(-m) + 1e-6), dtype=F))


def test_gates_are_capped():
    assert PV.soft_limit(torch.tensor(1e6, dtype=F), 3.0) == 3.0 and abs(PV.soft_limit(torch.tensor(0.01, dtype=F), 3.0) - 0.01) < 1e-6
    assert torch.allclose(PV.log_sigmoid(torch.tensor(-2.0, dtype=F)), torch.log(torch.sigmoid(torch.tensor(-2.0, dtype=F))))


def test_the_correction_chooses_and_does_not_weigh():
    s = torch.tensor([[0.9, 0.5, 0.4, 0.1]], dtype=F)
    idx, wt = PV.choose(s, torch.tensor([-1.0, 0.0, 0.0, 0.6], dtype=F), 2)
    assert idx.tolist() == [[3, 1]] and torch.allclose(wt, torch.tensor([[0.1, 0.5]], dtype=F))


def test_only_the_best_groups_take_part_also_with_negative_scores():
    s = torch.tensor([[0.9, 0.05, 0.5, 0.5, 0.6, 0.3]], dtype=F)
    c = torch.full((6,), -2.0, dtype=F)                        # every choice score is negative
    idx, _ = PV.choose(s, c, 2, {"count": 3, "keep": 1})       # sums 0.95, 1.0, 0.9: the middle group, not the best expert's
    assert idx.tolist() == [[2, 3]]
    idx, _ = PV.choose(s, c, 3, {"count": 3, "keep": 2})
    assert idx.tolist() == [[0, 2, 3]]
    idx, _ = PV.choose(s, c, 1, {"count": 6, "keep": 2})       # groups of one: their only score
    assert idx.tolist() == [[0]]
    three = torch.tensor([[0.9, 0.1, 0.8, 0.6, 0.6, 0.55]], dtype=F)
    idx, _ = PV.choose(three, torch.zeros(6, dtype=F), 1, {"count": 2, "keep": 1})   # the two largest of three: 1.7 against 1.2
    assert idx.tolist() == [[0]]


def test_the_sides_are_normed_before_half_of_their_sum():
    import helpers
    import kavotar_helpers as VH
    from atoma_infer_b200.weights.random_init import random_tensors

    cfg = VH.CONFIGS["U"][0]
    from atoma_infer_b200.config.registry import architecture
    from atoma_infer_b200.parts.model import declared_tensors

    arch = architecture("Kavotar")
    w = random_tensors(declared_tensors(arch.build_spec(arch.parse_config(cfg))), 3, std=0.05, norm_jitter=0.1, scales=VH.SCALES)
    x = rnd(11, cfg["width"])
    m = cfg["layers"][1]["mixer"]
    y = PV.parallel(m, w, "l1.mix.", x, 1e-5)
    loud = {k: (v * 64.0 if k in ("l1.mix.left.o", "l1.mix.right.o") else v) for k, v in w.items()}
    assert torch.allclose(PV.parallel(m, loud, "l1.mix.", x, 1e-12), PV.parallel(m, w, "l1.mix.", x, 1e-12), atol=1e-6)  # (a size the norm takes off)
    gone = dict(w, **{"l1.mix.left.out": w["l1.mix.left.out"] * 0})
    right = PV.rms(PV.token_mixing(m["right"], w, "l1.mix.right.", x, 1e-5), 1e-5) * w["l1.mix.right.out"].to(F)
    assert torch.allclose(PV.parallel(m, gone, "l1.mix.", x, 1e-5), 0.5 * right) and not torch.allclose(y, 0.5 * right)
    assert helpers.ROOT


@pytest.mark.parametrize("name", ["U", "V", "W"])
def test_a_longer_sequence_does_not_change_earlier_positions(name, tmp_path):
    import helpers
    import kavotar_helpers as VH

    cfg, _ = VH.CONFIGS[name]
    d = VH.make_model(str(tmp_path / "m"), name, seed=1)
    w = helpers.read_weights(d)
    toks = helpers.random_tokens(cfg["vocab"], (40,), seed=2)["r0"]
    assert torch.allclose(PV.forward(cfg, w, toks)[:23], PV.forward(cfg, w, toks[:23]), atol=1e-9)
