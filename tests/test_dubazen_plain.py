"""Dubazen without a GPU: the configuration reader, the description made of parts, the cache needs of its layers, random
weights around a part's own mean, the constants a layer of streams works out, and the plain implementation against
restatements of its mechanisms in other algebra."""
import copy
import math

import pytest
import torch

import plain_dubazen as pd
from dubazen_configs import DUBAZEN_A, DUBAZEN_B, DUBAZEN_C


def resolve(cfg, shapes=None):
    import ferrox_b200  # noqa: F401  (registers the architectures)
    from ferrox_b200.config.registry import resolve as r

    return r(cfg, shapes)


def test_configuration_is_read_layer_by_layer():
    cfg, spec = resolve(DUBAZEN_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale, cfg.streams) == (211, 64, 1e-5, 3.0, 2)
    m = cfg.layers[0].mixer
    a, r = m.left, m.right
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.rot_dims, a.rot_base) == (4, 2, 32, 48, 0.3, 16, 500.0)
    assert (r.heads, r.dim, r.vdim, r.decay) == (2, 16, 32, (0.7, 0.97)) and (m.left_scale, m.right_scale) == (0.8, 1.1)
    f = cfg.layers[0].mlp
    assert (f.experts, f.top, f.ff, f.limit, f.shared_ff, f.shared_limit) == (6, 2, 32, 1.5, 48, 0.9)
    assert cfg.layers[3].mlp.shared_ff == 0 and cfg.layers[2].mlp is None
    mm = cfg.layers[1].mixer
    assert (mm.inner, mm.state, mm.dt_rank, mm.conv) == (96, 16, 8, 4)
    g = cfg.layers[2].mixer
    assert (g.heads, g.dim, g.vdim, g.tau, g.decay_rank) == (4, 16, 32, 16.0, None)
    assert spec.streams == 2 and spec.embedding_scale == 3.0 and [(e.layer, e.cache) for e in spec.schedule] == [(i, i) for i in range(4)]
    left, right = spec.layers[0].mixer.mixers
    assert left.value_turn == (500.0, "halves") and left.rotated_norm_eps == 1e-5 and left.qkv_bias and left.o_bias and left.sink
    assert spec.layers[0].ffn.activation == ("clamped_swish", 1.5, 1.702) and spec.layers[0].ffn.shared_activation[1] == 0.9
    assert resolve(DUBAZEN_B)[1].layers[3].mixer.mixers[0].position is None      # no rotated dimensions; values turn all the same
    assert resolve(DUBAZEN_B)[1].layers[3].mixer.mixers[0].value_turn[0] == 33.0


def test_defaults_of_keys_that_may_be_absent():
    c = copy.deepcopy(DUBAZEN_A)
    for key in ("kv_heads", "vdim"):
        del c["layers"][0]["mixer"]["left"][key]
    del c["layers"][0]["mixer"]["right"]["vdim"], c["layers"][2]["mixer"]["vdim"], c["layers"][1]["mlp"], c["embedding"], c["streams"]
    c["layers"][0]["mlp"]["shared"] = None
    cfg, spec = resolve(c)
    m = cfg.layers[0].mixer
    assert (m.left.kv_heads, m.left.vdim, m.right.vdim, cfg.layers[2].mixer.vdim) == (4, 32, 16, 16)
    assert cfg.embedding_scale == 1.0 and cfg.streams == 1 and cfg.layers[1].mlp is None and cfg.layers[0].mlp.shared_ff == 0


@pytest.mark.parametrize("change,text", [
    (lambda c: c["layers"][0].update(type="ring"), "not implemented"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "not implemented"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(vdim=47), "vdim"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "exceeds"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=34), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mixer"].pop("dt_rank"), "dt_rank"),
    (lambda c: c["layers"][2]["mixer"].update(tau=0.0), "tau"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "empty"),
])
def test_configurations_that_are_refused(change, text):
    from ferrox_b200 import ConfigError

    cfg = copy.deepcopy(DUBAZEN_A)
    change(cfg)
    with pytest.raises(ConfigError, match=text):
        resolve(cfg)


def test_more_streams_than_the_kernel_holds_are_refused():
    from ferrox_b200.parts.build import build_model

    with pytest.raises(ValueError, match="streams"):
        build_model(resolve(dict(DUBAZEN_A, streams=9))[1])


def test_description_declares_the_tensors_and_the_cache_needs():
    from ferrox_b200.parts.build import build_model

    _, spec = resolve(DUBAZEN_A, {"l2.mix.a1": (9, 64)})      # the decay's inner width: its tensor's shape
    model = build_model(spec)
    decls = {d.name: d for d in model.tensor_decls()}
    shape = {n: d.shape for n, d in decls.items()}
    assert shape["embed"] == (211, 64) and shape["head"] == (211, 64) and shape["final.norm"] == ()
    assert shape["l0.norm1"] == shape["l0.norm2"] == () and shape["l0.hc1.in"] == shape["l0.hc2.out"] == (2,)
    assert shape["l0.hc1.mix"] == (2, 2)
    p = "l0.mix.left."
    assert shape[p + "q"] == (128, 64) and shape[p + "k"] == (64, 64) and shape[p + "v"] == (96, 64) and shape[p + "v.b"] == (96,)
    assert shape[p + "g"] == (192, 64) and shape[p + "o"] == (64, 192) and shape[p + "o.b"] == (64,) and shape[p + "sink"] == (4,)
    p = "l0.mix.right."
    assert shape[p + "q"] == (32, 64) and shape[p + "v"] == (64, 64) and shape[p + "norm"] == (64,) and shape[p + "o"] == (64, 64)
    p = "l1.mix."
    assert shape[p + "in"] == (192, 64) and shape[p + "conv"] == (96, 4) and shape[p + "x"] == (40, 96) and shape[p + "dt"] == (96, 8)
    assert shape[p + "A_log"] == (96, 16) and shape[p + "D"] == shape[p + "dt.b"] == shape[p + "conv.b"] == (96,)
    p = "l2.mix."
    assert shape[p + "a1"] == (9, 64) and shape[p + "a2"] == (64, 9) and shape[p + "a2.b"] == (64,) and shape[p + "norm"] == (32,)
    assert shape["l0.mlp.router"] == (6, 64) and shape["l0.mlp.shared.down"] == (64, 48) and "l3.mlp.shared.up" not in shape
    # a layer without a feed-forward needs neither norm nor connections for it; a checkpoint may carry them all the same
    assert all(decls["l2." + n].optional for n in ("norm2", "hc2.in", "hc2.out", "hc2.mix")) and not decls["l2.hc1.mix"].optional
    caches = model.cache_specs()
    assert [t.token_shape for t in caches[0].paged.tensors] == [(2, 32), (2, 48)]
    assert caches[0].state.parts == (("1.matrix", (2, 32, 16)),)
    assert caches[1].paged is None and caches[1].state.parts == (("matrix", (96, 16)), ("conv_tail", (3, 96)))
    assert caches[2].state.parts == (("matrix", (4, 16, 32)),)
    assert model.graph_safe()


def test_random_weights_lie_around_a_parts_own_mean():
    from ferrox_b200.parts.build import build_model
    from ferrox_b200.weights.random_init import random_tensors

    w = dict(random_tensors(build_model(resolve(DUBAZEN_B)[1]).tensor_decls(), 3, torch.float32, 0.05, "ones"))
    assert float((w["l1.hc1.mix"] - torch.eye(5)).abs().max()) < 0.25 and float(w["l1.hc1.mix"].std()) > 0.1
    assert abs(float(w["l1.hc2.in"].mean()) - 0.2) < 0.1 and abs(float(w["l1.hc2.out"].mean()) - 1.0) < 0.1
    assert abs(float(w["l2.mix.dt.b"].mean()) + 3.0) < 0.1 and abs(float(w["l2.mix.D"].mean()) - 1.0) < 0.1
    assert abs(float(w["l2.mix.o"].mean())) < 0.01 and float(w["final.norm"]) == 1.0


def test_a_layer_of_streams_works_out_its_constants():
    """Two updates with a reading between them, one after the other, against the one update and the one reading that the
    block's constants describe."""
    from ferrox_b200.parts.base import Runtime, build_part
    from ferrox_b200.parts.specs import HyperBlockSpec, NormSpec, PlainMlpSpec, SelectiveScanSpec, StreamNormSpec
    from ferrox_b200.parts import build  # noqa: F401  (registers the built-in parts)
    from ferrox_b200.weights import loader as wl
    from ferrox_b200.weights.random_init import random_tensors

    S, W = 3, 8
    norm = lambda q: StreamNormSpec(NormSpec(W, 1e-5, "", name=f"n{q}", scalar=True), S, f"in{q}")
    spec = HyperBlockSpec(norm1=norm(1), mixer=SelectiveScanSpec(W, 4, 2, 2, 2, "m."), norm2=norm(2), ffn=PlainMlpSpec(W, 4, "f."),
                          streams=S, connections=(("mix1", "out1"), ("mix2", "out2")))
    block = build_part(spec)
    w = dict(random_tensors(block.tensor_decls(), 5, torch.float32, 0.4, "around_one"))
    block.load(wl.from_dict(w, block.tensor_decls(), "cpu", torch.float32), Runtime(torch.device("cpu"), torch.float32))
    g = torch.Generator().manual_seed(1)
    X, y1, y2 = torch.randn(S, 5, W, generator=g), torch.randn(5, W, generator=g), torch.randn(5, W, generator=g)
    A = pd.mix_streams(X, y1, w["mix1"], w["out1"])
    u2 = pd.read_streams(A, w["in2"])
    B = pd.mix_streams(A, y2, w["mix2"], w["out2"])
    t = lambda v: torch.as_tensor(v, dtype=torch.float32)
    got_u2 = torch.einsum("snw,s->nw", X, t(block.mid_reads)) + block.mid_result[0] * y1
    got_B = (torch.einsum("snw,st->tnw", X, t(block.mix)) + t(block.out1)[:, None, None] * y1 + t(block.out2)[:, None, None] * y2)
    assert torch.allclose(got_u2, u2, atol=1e-5) and torch.allclose(got_B, B, atol=1e-5)


def test_values_pairs_come_together():
    from ferrox_b200.parts.base import build_part
    from ferrox_b200.parts.specs import AttentionSpec
    from ferrox_b200.parts import build  # noqa: F401  (registers the built-in parts)

    kw = dict(hidden=16, n_heads=2, n_kv_heads=1, head_dim=8, value_dim=6, qkv_bias=False, position=None, window=None, prefix="m.")
    a = build_part(AttentionSpec(**kw, value_turn=(100.0, "halves")))
    assert a._pairs_together(2, "cpu").tolist() == [0, 3, 1, 4, 2, 5, 6, 9, 7, 10, 8, 11]
    assert build_part(AttentionSpec(**kw, value_turn=(100.0, "adjacent")))._pairs_together(2, "cpu") is None
    assert build_part(AttentionSpec(**kw))._pairs_together(2, "cpu") is None
    for bad in (dict(value_dim=5), dict(value_turn=(100.0, "odd"))):
        with pytest.raises(ValueError):
            build_part(AttentionSpec(**dict(dict(kw, value_turn=(100.0, "halves")), **bad)))


# ------------------------------------------------------------------ the plain implementation, restated
def test_plain_rotation_is_a_complex_product_and_turns_back():
    g = torch.Generator().manual_seed(1)
    x = torch.randn(30, 3, 14, generator=g, dtype=torch.float64)
    got = pd.turn_halves(x, 10, 50.0)
    for p in (0, 1, 17, 29):
        for i in range(5):
            z = torch.complex(x[p, :, i], x[p, :, i + 5]) * torch.exp(torch.tensor(1j * p * 50.0 ** (-2 * i / 10)))
            assert torch.allclose(got[p, :, i], z.real, atol=1e-5) and torch.allclose(got[p, :, i + 5], z.imag, atol=1e-5)
    assert torch.equal(got[:, :, 10:], x[:, :, 10:])
    assert torch.allclose(pd.turn_halves(got, 10, 50.0, -1.0), x, atol=1e-6)


def test_plain_turned_values_depend_on_the_distance_alone():
    """What a query makes of a value hangs on how far away it is: the value turned by minus the distance."""
    n, V, base = 12, 6, 30.0
    v = torch.randn(n, 1, V, generator=torch.Generator().manual_seed(2), dtype=torch.float64)
    turned = pd.turn_halves(v, V, base)
    for i, j in ((11, 0), (7, 5), (4, 4)):
        o = torch.zeros(n, 1, V, dtype=torch.float64)
        o[i] = turned[j]
        back = pd.turn_halves(o, V, base, -1.0)[i]
        moved = torch.zeros(i - j + 1, 1, V, dtype=torch.float64)
        moved[i - j] = v[j]
        assert torch.allclose(back, pd.turn_halves(moved, V, base, -1.0)[i - j], atol=1e-5)


def test_plain_recurrences_as_sums_over_the_past():
    g = torch.Generator().manual_seed(3)
    R = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64) * 0.5
    n, W = 9, 7
    # linear attention with a decay per key channel
    H, D, V, r = 2, 3, 4, 2
    w = {"q": R(H * D, W), "k": R(H * D, W), "v": R(H * V, W), "g": R(H * V, W), "o": torch.eye(H * V, dtype=torch.float64),
         "norm": R(V) + 1, "a1": R(r, W), "a2": R(H * D, r), "a2.b": R(H * D)}
    h = R(n, W)
    got = pd.gated_linear_attention(h, w, "", {"heads": H, "dim": D, "vdim": V, "tau": 3.0}, 1e-5)
    z = h @ w["a1"].T @ w["a2"].T + w["a2.b"]
    log_a = (torch.nn.functional.logsigmoid(z) / 3.0).cumsum(0).view(n, H, D)
    q, k, v = (h @ w["q"].T / math.sqrt(D)).view(n, H, D), (h @ w["k"].T).view(n, H, D), (h @ w["v"].T).view(n, H, V)
    for t in range(n):
        o = sum((q[t] * k[s] * torch.exp(log_a[t] - log_a[s])).sum(-1, keepdim=True) * v[s] for s in range(t + 1))
        o = (o / torch.sqrt((o * o).mean(-1, keepdim=True) + 1e-5) * w["norm"]).reshape(-1)
        assert torch.allclose(got[t], o * torch.nn.functional.silu(h[t] @ w["g"].T), atol=1e-10)
    # the selective state space
    I, N, K = 5, 3, 3
    w = {"in": R(2 * I, W), "conv": R(I, K), "conv.b": R(I), "x": R(2 + 2 * N, I), "dt": R(I, 2), "dt.b": R(I), "A_log": R(I, N),
         "D": R(I), "o": torch.eye(I, dtype=torch.float64)}
    got = pd.selective_scan(h, w, "", {"inner": I, "state": N, "dt_rank": 2, "conv": K}, 1e-5)
    xz = h @ w["in"].T
    x = torch.nn.functional.conv1d(xz[:, :I].T[None], w["conv"][:, None], w["conv.b"], padding=K - 1, groups=I)[0, :, :n].T
    x = torch.nn.functional.silu(x)
    low = x @ w["x"].T
    dt = torch.nn.functional.softplus(low[:, :2] @ w["dt"].T + w["dt.b"])
    cum = dt.cumsum(0)
    for t in range(n):
        y = w["D"] * x[t]
        for s in range(t + 1):
            decay = torch.exp(-(cum[t] - cum[s])[:, None] * torch.exp(w["A_log"]))
            y = y + (decay * (dt[s] * x[s])[:, None] * low[s, 2:2 + N] * low[t, 2 + N:]).sum(1)
        assert torch.allclose(got[t], y * torch.nn.functional.silu(xz[t, I:]), atol=1e-10)
    # one fixed decay a head
    w = {"q": R(2 * 3, W), "k": R(2 * 3, W), "v": R(2 * 2, W), "g": R(4, W), "o": torch.eye(4, dtype=torch.float64), "norm": R(4)}
    got = pd.fixed_decay_attention(h, w, "", {"heads": 2, "dim": 3, "vdim": 2, "decay": [0.5, 0.9]}, 1e-5)
    s = torch.nn.functional.silu
    q, k, v = s(h @ w["q"].T).view(n, 2, 3), s(h @ w["k"].T).view(n, 2, 3), s(h @ w["v"].T).view(n, 2, 2)
    d = torch.tensor([0.5, 0.9], dtype=torch.float64)[:, None]
    for t in range(n):
        o = sum((q[t] * k[u]).sum(-1, keepdim=True) * d ** (t - u) * v[u] for u in range(t + 1)).reshape(-1)
        o = o / torch.sqrt((o * o).mean() + 1e-5) * w["norm"]
        assert torch.allclose(got[t], o * torch.sigmoid(h[t] @ w["g"].T), atol=1e-10)


def test_plain_experts_and_sinks():
    W = {"gate": torch.tensor([[3.0], [-1.0]]), "up": torch.tensor([[-5.0], [0.5]]), "down": torch.tensor([[1.0, 2.0]])}
    swish = lambda v: v / (1 + math.exp(-1.702 * v))
    assert abs(float(pd.expert(W, "", torch.tensor([[1.0]]), 2.0)) - (swish(2.0) * (-2.0 + 1) + 2 * swish(-1.0) * 1.5)) < 1e-5
    s = torch.tensor([[0.3, -1.0], [2.0, 0.7]])
    w = pd.softmax_with_sink(s, torch.tensor(0.9))
    den = math.exp(2.0) + math.exp(0.7) + math.exp(0.9)
    assert torch.allclose(w[1], torch.tensor([math.exp(2.0) / den, math.exp(0.7) / den]))
    assert torch.allclose(w[0], torch.tensor([math.exp(0.3) / (math.exp(0.3) + math.exp(0.9)), 0.0]))


def test_every_mechanism_shows_in_the_logits():
    """The logits of configurations move when any one mechanism is changed: what the comparisons with the engine rest on."""
    from ferrox_b200.parts.build import build_model
    from ferrox_b200.weights.random_init import random_tensors

    decls = build_model(resolve(DUBAZEN_A)[1]).tensor_decls()
    W = {n: t.float() for n, t in random_tensors(decls, 61, torch.bfloat16, 0.15, "around_one")}
    toks = [(7 * i * i + 3) % 211 for i in range(60)]
    want = pd.forward(DUBAZEN_A, W, toks)

    def moved(cfg=DUBAZEN_A, w=W):
        return float((pd.forward(cfg, w, toks) - want).abs().max() / want.abs().max())

    def changed(f):
        c = copy.deepcopy(DUBAZEN_A)
        f(c)
        return moved(c)

    assert changed(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=14)) > 1e-3
    assert changed(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(base=400.0)) > 1e-3
    assert changed(lambda c: c["layers"][0]["mixer"]["left"].update(scale=0.4)) > 1e-3
    assert changed(lambda c: c["layers"][0]["mixer"].update(left_scale=0.9)) > 1e-3
    assert changed(lambda c: c["layers"][3]["mixer"].update(right_scale=0.4)) > 1e-3
    assert changed(lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.7, 0.9])) > 1e-3
    assert changed(lambda c: c["layers"][2]["mixer"].update(tau=8.0)) > 1e-3
    assert changed(lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.3)) > 1e-3
    assert changed(lambda c: c["layers"][0]["mlp"]["shared"].update(limit=0.3)) > 1e-3
    assert changed(lambda c: c["embedding"].update(scale=2.0)) > 1e-3
    for name in ("l0.mix.left.sink", "l0.mix.left.q.b", "l0.mix.left.v.b", "l0.mix.left.o.b", "l0.mix.left.g", "l1.mix.conv.b",
                 "l1.mix.dt.b", "l1.mix.A_log", "l1.mix.D", "l2.mix.a2.b", "l2.mix.norm", "l0.hc1.mix", "l0.hc2.mix", "l1.hc2.out",
                 "l2.hc1.in", "l0.norm2", "final.norm", "l0.mlp.shared.up", "l0.mix.right.norm"):
        assert moved(w=dict(W, **{name: W[name] * -0.5})) > 1e-4, name
