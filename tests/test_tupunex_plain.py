"""The plain Tupunex implementation, mechanism by mechanism, against what each must do."""
import math

import pytest
import torch

import plain_tupunex as PX
import tupunex_helpers as XH

F = torch.float64


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F)


def test_norm_has_eps_inside_the_root():
    x, w = torch.tensor([[1.0, 3.0, 5.0, 7.0]], dtype=F), torch.tensor([1.0, 2.0, 1.0, 0.5], dtype=F)
    assert torch.allclose(PX.rms_norm(x, w, 0.25), x / math.sqrt(21.0 + 0.25) * w)


def test_streams_are_mixed_from_the_old_ones_by_from_and_to():
    X, y = rnd(4, 3, 5), rnd(4, 5, seed=1)
    M, b = torch.tensor([[1.0, 0.5, 0.0], [0.0, 2.0, -1.0], [0.25, 0.0, 1.0]], dtype=F), torch.tensor([0.0, 1.0, -2.0], dtype=F)
    Y = PX.mix_streams(X, M, b, y)
    assert torch.allclose(Y[:, 0], X[:, 0] + 0.25 * X[:, 2])                  # what flows INTO stream 0: the matrix' first column
    assert torch.allclose(Y[:, 1], 0.5 * X[:, 0] + 2.0 * X[:, 1] + y)
    assert torch.allclose(Y[:, 2], -X[:, 1] + X[:, 2] - 2.0 * y)
    assert torch.allclose(PX.read_streams(X, torch.tensor([1.0, 0.0, 3.0], dtype=F)), X[:, 0] + 3.0 * X[:, 2])


def test_convolution_is_causal_and_starts_from_zeros():
    u, w = rnd(7, 2), rnd(2, 3, seed=1)
    y = PX.causal_conv(u, w)
    assert torch.allclose(y[0], w[:, 2] * u[0]) and torch.allclose(y[1], w[:, 1] * u[0] + w[:, 2] * u[1])
    assert torch.allclose(y[5], w[:, 0] * u[3] + w[:, 1] * u[4] + w[:, 2] * u[5])
    assert torch.allclose(PX.causal_conv(u, w[:, 2:]), w[:, 2] * u)


def test_a_bias_enters_before_the_convolution_and_not_before_the_start():
    """The row of a request's first token sees its own bias once, not the bias of rows that do not exist."""
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 4, "scale": 1.0, "diff": 0.2, "conv": 2}
    w = {"q": rnd(4, 3), "k": rnd(4, 3, seed=1), "v": torch.zeros(4, 3, dtype=F), "g": torch.zeros(1, 3, dtype=F), "o": torch.eye(4, dtype=F),
         "q.b": torch.zeros(4, dtype=F), "k.b": torch.zeros(4, dtype=F), "v.b": torch.tensor([1.0, 2.0, 0.0, -1.0], dtype=F)}
    w.update({x + ".conv": torch.ones(4, 2, dtype=F) for x in "qk"}, **{"v.conv": torch.tensor([[3.0, 1.0]] * 4, dtype=F)})
    w.update({x: torch.zeros(2, dtype=F) for x in ("lq1", "lk1", "lq2", "lk2")})
    seen = []
    keep = PX.two_maps
    try:
        PX.two_maps = lambda q, k, v, *a: seen.append(v) or keep(q, k, v, *a)
        PX.differential_attention(m, w, "", rnd(3, 3, seed=2), 1e-5)
    finally:
        PX.two_maps = keep
    assert torch.allclose(seen[0][0, 0], w["v.b"]) and torch.allclose(seen[0][1, 0], 4.0 * w["v.b"])


def test_a_window_keeps_itself_and_what_lies_less_than_its_size_back():
    see = PX.visible(10, 4)
    assert see[9].nonzero().flatten().tolist() == [6, 7, 8, 9] and see[2].nonzero().flatten().tolist() == [0, 1, 2]
    assert PX.visible(5)[4].all() and not PX.visible(5)[1, 2]


def test_each_map_is_an_attention_of_its_own_over_the_same_values():
    q, k, v = rnd(5, 4, 2, 3), rnd(5, 2, 2, 3, seed=1), rnd(5, 2, 6, seed=2)
    a = PX.two_maps(q, k, v, 0.7, None, PX.visible(5))
    for h, m in ((0, 0), (1, 1), (3, 0)):
        p = torch.softmax(0.7 * q[4, h, m] @ k[:, h // 2, m].T, 0)       # head h reads key/value head h // 2
        assert torch.allclose(a[4, h, m], p @ v[:, h // 2])
    assert torch.allclose(a[0, 3, 1], v[0, 1])
    capped = PX.two_maps(q * 50.0, k, v, 0.7, 0.5, PX.visible(5))
    s = 0.5 * torch.tanh(0.7 * 50.0 * q[3, 2, 1] @ k[:4, 1, 1].T / 0.5)
    assert torch.allclose(capped[3, 2, 1], torch.softmax(s, 0) @ v[:4, 1])


def test_the_difference_is_normed_over_a_heads_values_and_scaled():
    a = rnd(3, 2, 2, 4)
    o = PX.difference(a, 0.3, 0.25, 0.5)
    d = a[1, 1, 0] - 0.3 * a[1, 1, 1]
    assert torch.allclose(o[1, 1], 0.75 * d / math.sqrt(float((d * d).mean()) + 0.5))
    w = {"lq1": torch.tensor([1.0, 2.0]), "lk1": torch.tensor([0.5, 0.25]), "lq2": torch.tensor([-1.0, 1.0]), "lk2": torch.tensor([1.0, 0.5])}
    assert abs(float(PX.map_weight(w, "", 0.4)) - (math.exp(1.0) - math.exp(-0.5) + 0.4)) < 1e-12


def test_a_gate_is_one_number_per_head():
    o, h, w = rnd(3, 2, 4), rnd(3, 5, seed=1), rnd(2, 5, seed=2)
    g = PX.gate_heads(o, h, w)
    assert torch.allclose(g[2, 1], o[2, 1] / (1.0 + math.exp(-float(h[2] @ w[1]))))


def test_rotation_pairs_the_halves_and_leaves_the_tail():
    x = rnd(9, 2, 10)
    y = PX.rotate_halves(x, 6, 100.0)
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.allclose(y[0], x[0])
    p, i = 7, 2
    a = p * 100.0 ** (-2.0 * i / 6)
    assert torch.allclose(y[p, 1, i], x[p, 1, i] * math.cos(a) - x[p, 1, i + 3] * math.sin(a))
    assert torch.allclose(y[p, 1, i + 3], x[p, 1, i + 3] * math.cos(a) + x[p, 1, i] * math.sin(a))
    assert torch.equal(PX.rotate_halves(x, 0, 100.0), x) and PX.rotate_halves(x[:, 0], 4, 10.0).shape == (9, 10)


def test_latent_attention_scores_both_parts_and_shares_the_rotated_key():
    m = {"heads": 2, "dim": 3, "rot_dim": 2, "vdim": 4, "kv_rank": 5, "scale": 0.6, "rot": {"dims": 2, "base": 10.0}}
    w = {"q": rnd(10, 6), "dkv": rnd(7, 6, seed=1), "dkv.norm": rnd(5, seed=2), "uk": rnd(6, 5, seed=3), "uv": rnd(8, 5, seed=4),
         "g": torch.zeros(2, 6, dtype=F), "o": torch.eye(8, dtype=F)}
    h = rnd(4, 6, seed=5)
    y = PX.latent_attention(m, w, "", h, 1e-5).reshape(4, 2, 4) * 2.0     # (a gate of zero halves)
    c = PX.rms_norm(h @ w["dkv"][:5].T, w["dkv.norm"], 1e-5)
    turn = lambda v: PX.rotate_halves(v, 2, 10.0)  # noqa: E731
    kr, q = turn(h @ w["dkv"][5:].T), (h @ w["q"].T).reshape(4, 2, 5)
    a = 1
    s = 0.6 * ((c @ w["uk"].T)[:, 3:] @ q[3, a, :3] + kr @ turn(q[:, a, 3:])[3])
    assert torch.allclose(y[3, a], torch.softmax(s, 0) @ (c @ w["uv"].T)[:, 4:])


def test_the_order_of_the_layers_repeats_a_stretch():
    assert PX.layer_runs({"layers": [0] * 5, "loop": {"start": 1, "stop": 3, "times": 3}}) == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert PX.layer_runs({"layers": [0] * 2}) == [0, 1]


@pytest.mark.parametrize("name", list(XH.CONFIGS))
def test_later_tokens_change_nothing_before_them(name, tmp_path):
    import helpers

    cfg, _ = XH.CONFIGS[name]
    w = helpers.read_weights(XH.make_model(str(tmp_path), name, seed=2))
    toks = helpers.random_tokens(cfg["vocab"], (24,), seed=1)["r0"]
    whole, part = PX.forward(cfg, w, toks), PX.forward(cfg, w, toks[:15])
    assert torch.allclose(whole[:15], part, atol=1e-9)
    other = PX.forward(cfg, w, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])  # the first token is still heard at the end
    assert float((other[-1] - whole[-1]).abs().max()) > 1e-4 * float(whole[-1].abs().max())
