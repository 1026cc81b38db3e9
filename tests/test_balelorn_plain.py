"""Balelorn without a GPU: the configuration reader, the description made of parts, the cache needs of its layers and
what a chunk gives back, the random tables, and the plain implementation against restatements of its mechanisms in
other algebra."""
import copy
import math

import pytest
import torch

import plain_balelorn as pb
from balelorn_configs import BALELORN_A, BALELORN_B, BALELORN_C


def resolve(cfg):
    import ferrox_b200  # noqa: F401  (registers the architectures)
    from ferrox_b200.config.registry import resolve as r

    return r(cfg)


def test_configuration_is_read_layer_by_layer():
    cfg, spec = resolve(BALELORN_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps) == (211, 64, 1e-5)
    a = cfg.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk, a.v_mix) == (4, 2, 32, 48, 0.2, 24, False)
    assert (a.rot.dims, a.rot.base) == (16, 500.0)
    f = cfg.layers[0].mlp
    assert (f.experts, f.top, f.ff, f.limit) == (6, 2, 32, 1.5) and cfg.layers[1].mlp.ff == 96
    assert cfg.layers[3].mlp is None
    assert [(e.layer, e.cache) for e in spec.schedule] == [(i, i) for i in range(4)]
    mixes = [b.mixer.value_mix for b in spec.layers]
    assert mixes[0] is None and mixes[1].source and not mixes[2].source and not mixes[3].source
    assert [b.mixer.chunk for b in spec.layers] == [24, 21, 24, 50]
    assert spec.layers[3].ffn is None and spec.layers[3].post2 is None
    cfgB, specB = resolve(BALELORN_B)
    assert cfgB.layers[1].mixer.chunk is None and cfgB.layers[2].mixer.rot is None
    assert specB.layers[0].mixer.value_mix.source and specB.layers[2].mixer.value_mix is None


def test_defaults_of_keys_that_may_be_absent():
    c = copy.deepcopy(BALELORN_B)
    for key in ("kv_heads", "vdim", "v_mix"):
        del c["layers"][2]["mixer"][key]
    del c["layers"][1]["mlp"]
    c["layers"][2]["mixer"]["mask"] = None
    c["layers"][2]["mixer"]["rot"] = {"dims": 0, "base": 10.0}
    m = resolve(c)[0].layers[2].mixer
    assert (m.kv_heads, m.vdim, m.v_mix, m.chunk, m.rot) == (2, 24, False, None, None)


@pytest.mark.parametrize("change,text", [
    (lambda c: c["layers"][0].update(type="ring"), "not implemented"),
    (lambda c: c["layers"][1]["mlp"].update(kind="gated"), "not implemented"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "exceeds"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=34), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"].update(mask=5), "object"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=16), "cannot be mixed"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "empty"),
])
def test_configurations_that_are_refused(change, text):
    from ferrox_b200 import ConfigError

    cfg = copy.deepcopy(BALELORN_A)
    change(cfg)
    with pytest.raises(ConfigError, match=text):
        resolve(cfg)


def test_description_declares_the_tensors_and_the_cache_needs():
    from ferrox_b200.parts.build import build_model

    _, spec = resolve(BALELORN_A)
    model = build_model(spec)
    decls = {d.name: d for d in model.tensor_decls()}
    shape = {n: d.shape for n, d in decls.items()}
    assert shape["embed"] == (211, 64) and shape["embed.norm"] == (64,) and shape["head"] == (211, 64)
    assert shape["l0.mix.q"] == (128, 64) and shape["l0.mix.k"] == (64, 64) and shape["l0.mix.v"] == (96, 64)
    assert shape["l0.mix.g"] == (192, 64) and shape["l0.mix.o"] == (64, 192) and shape["l0.mix.sink"] == (4,)
    assert "l0.mix.vmix" not in shape and shape["l1.mix.vmix"] == () and shape["l2.mix.vmix"] == ()
    assert decls["l1.mix.vmix"].optional and not decls["l2.mix.vmix"].optional      # (the source's is never read)
    assert shape["l0.mlp.table"] == (211, 2) and decls["l0.mlp.table"].integer and decls["l0.mlp.table"].below == 6
    assert shape["l0.mlp.e5.down"] == (64, 32) and shape["l1.mlp.gate"] == (96, 64)
    for n in ("norm1", "norm1b", "ls1", "norm2", "norm2b", "ls2"):
        assert shape["l2." + n] == (64,)
    # a layer without a feed-forward needs no norms for it; a checkpoint may carry them all the same
    assert not decls["l3.ls1"].optional and all(decls["l3." + n].optional for n in ("norm2", "norm2b", "ls2"))
    caches = model.cache_specs()
    assert [t.token_shape for t in caches[0].paged.tensors] == [(2, 32), (2, 48)]
    assert [c.paged.chunk for c in caches] == [24, 21, 24, 50] and all(c.paged.window is None for c in caches)
    assert model.graph_safe()
    assert [t.token_shape for t in build_model(resolve(BALELORN_C)[1]).cache_specs()[2].paged.tensors] == [(3, 96), (3, 40)]


def test_a_chunk_gives_its_pages_back_when_the_request_leaves_it():
    """Chunks of 10 positions on pages of 4: after every step the request holds exactly the pages that the chunk of its
    next position has begun, whatever the portions; a group without chunks keeps everything."""
    from ferrox_b200.cache.manager import CacheManager
    from ferrox_b200.cache.specs import CacheSpec, KvCacheSpec

    specs = [CacheSpec(paged=KvCacheSpec(1, 4, chunk=10)), CacheSpec(paged=KvCacheSpec(1, 4)),
             CacheSpec(paged=KvCacheSpec(1, 4, chunk=10)), CacheSpec(paged=KvCacheSpec(1, 4, chunk=7))]
    for portions in ([1] * 60, [7, 2, 11, 3, 30, 1, 6], [60]):
        m = CacheManager(specs, page_size=4, n_pages=32, max_slots=2, max_positions=64, device="cpu", dtype=torch.float32)
        assert set(m.groups) == {("chunk", 10), None, ("chunk", 7)} and m.groups[("chunk", 10)].caches == [0, 2]
        slot, n = m.open_request(), 0
        for add in portions:
            assert m.reserve_step([slot], [add]) is not None
            n += add
            m.commit_step([slot], [add])
            m.check_invariants()
            held = m.held_pages(slot)
            for size in (10, 7):
                first, last = n // size * size // 4, -(-n // 4)
                assert len(held[("chunk", size)]) == max(0, last - first), (size, n)
            assert len(held[None]) == -(-n // 4)
            assert m.layer_cache(0).chunk == 10 and m.layer_cache(1).chunk is None
        m.close_request(slot)
        m.check_invariants()
        assert all(free == 32 for free in m.free_pages().values())


def test_a_chunk_goes_without_a_window():
    from ferrox_b200.cache.manager import CacheError, CacheManager
    from ferrox_b200.cache.specs import CacheSpec, KvCacheSpec

    for bad in (KvCacheSpec(1, 4, window=8, chunk=10), KvCacheSpec(1, 4, chunk=0)):
        with pytest.raises(CacheError, match="chunk"):
            CacheManager([CacheSpec(paged=bad)], page_size=4, n_pages=4, max_slots=1, max_positions=64, device="cpu",
                         dtype=torch.float32)


def test_prompt_work_items_begin_at_the_chunk():
    from ferrox_b200.kernels import ops

    assert [ops.first_key(p, None, 100) for p in (0, 99, 100, 250)] == [0, 0, 100, 200]
    assert ops.first_key(250, 20, None) == 231 and ops.first_key(250, 20, 100) == 231 and ops.first_key(205, 20, 100) == 200
    items, merges, parts = ops.prefill_tc_plan([(1000, 0), (3, 777)], None, 8, run_blocks=0, chunk=300)
    seen = {}
    for tok0, rows, entry, pos0, kb, end, part, _ in items.tolist():
        assert part == -1 and kb == pos0 // 300 * 300 // 128 and end == (pos0 + rows - 1) // 128 + 1
        seen[(entry, tok0)] = rows
    assert not len(merges) and parts == 0 and sum(seen.values()) == 1003


def test_random_tables_name_different_experts_everywhere():
    from ferrox_b200.weights.random_init import distinct_rows

    t = distinct_rows(123, (500, 3), 7)
    assert t.dtype == torch.int32 and int(t.min()) == 0 and int(t.max()) == 6
    assert all(len(set(r)) == 3 for r in t.tolist()) and len({tuple(r) for r in t.tolist()}) > 100
    assert torch.equal(distinct_rows(123, (40, 3), 7), t[:40])         # a row does not depend on how many there are
    assert not torch.equal(distinct_rows(124, (500, 3), 7), t)
    assert sorted(distinct_rows(5, (1, 4), 4)[0].tolist()) == [0, 1, 2, 3]
    with pytest.raises(ValueError):
        distinct_rows(5, (1, 5), 4)


# ------------------------------------------------------------------ the plain implementation, restated
def test_plain_rotation_is_a_complex_product():
    g = torch.Generator().manual_seed(1)
    x = torch.randn(30, 3, 14, generator=g, dtype=torch.float64)
    got = pb.rotate_halves(x, 10, 50.0)
    for p in (0, 1, 17, 29):
        for i in range(5):
            z = torch.complex(x[p, :, i], x[p, :, i + 5]) * torch.exp(torch.tensor(1j * p * 50.0 ** (-2 * i / 10)))
            assert torch.allclose(got[p, :, i], z.real, atol=1e-5) and torch.allclose(got[p, :, i + 5], z.imag, atol=1e-5)
    assert torch.equal(got[:, :, 10:], x[:, :, 10:])


def test_plain_chunks_sinks_values_gate_and_experts():
    m = pb.chunk_mask(9, 4)
    assert m.int().sum(dim=1).tolist() == [1, 2, 3, 4, 1, 2, 3, 4, 1] and pb.chunk_mask(9, None).sum() == 45
    s = torch.tensor([[0.3, -1.0], [2.0, 0.7]])
    w = pb.softmax_with_sink(s, pb.chunk_mask(2, None), torch.tensor(0.9))
    den = math.exp(2.0) + math.exp(0.7) + math.exp(0.9)
    assert torch.allclose(w[1], torch.tensor([math.exp(2.0) / den, math.exp(0.7) / den]))
    assert torch.allclose(w[0], torch.tensor([math.exp(0.3) / (math.exp(0.3) + math.exp(0.9)), 0.0]))
    a, b = torch.randn(5), torch.randn(5)
    assert torch.allclose(pb.mixed_values(a, b, 0.25), a + 0.25 * (b - a))
    z = torch.linspace(-4, 4, 33)
    assert torch.allclose(pb.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-6)
    W = {"e.gate": torch.tensor([[3.0], [-1.0]]), "e.up": torch.tensor([[-5.0], [0.5]]), "e.down": torch.tensor([[1.0, 2.0]])}
    y = pb.expert(W, "e.", torch.tensor([[1.0]]), 2.0)
    swish = lambda v: v / (1 + math.exp(-1.702 * v))
    assert abs(float(y) - (swish(2.0) * (-2.0 + 1) + 2 * swish(-1.0) * 1.5)) < 1e-5


def test_every_mechanism_shows_in_the_logits():
    """The logits of configuration A move when any one mechanism is changed: what the comparisons with the engine rest on."""
    import ferrox_b200  # noqa: F401
    from ferrox_b200.parts.build import build_model
    from ferrox_b200.weights.random_init import random_tensors

    decls = build_model(resolve(BALELORN_A)[1]).tensor_decls()
    W = {n: t.float() if t.is_floating_point() else t.long() for n, t in random_tensors(decls, 51, torch.bfloat16, 0.2, "around_one")}
    toks = [(7 * i * i + 3) % 211 for i in range(60)]
    want = pb.forward(BALELORN_A, W, toks)

    def moved(cfg=BALELORN_A, w=W):
        return float((pb.forward(cfg, w, toks) - want).abs().max() / want.abs().max())

    def with_mixer(i, **kw):
        c = copy.deepcopy(BALELORN_A)
        c["layers"][i]["mixer"].update(kw)
        return c

    assert moved(with_mixer(0, mask={"size": 25})) > 1e-3 and moved(with_mixer(0, mask=None)) > 1e-3
    assert moved(with_mixer(1, rot={"dims": 46, "base": 10000.0})) > 1e-3 and moved(with_mixer(0, rot={"dims": 16, "base": 400.0})) > 1e-3
    assert moved(with_mixer(2, v_mix=False)) > 1e-3 and moved(with_mixer(0, scale=0.25)) > 1e-3
    for name, factor in (("l0.mix.sink", 0.0), ("l0.mix.g", -1.0), ("l3.mix.vmix", 0.0), ("l0.ls1", 1.3), ("l0.ls2", 1.3),
                         ("l1.norm2b", 1.3), ("embed.norm", 1.5)):
        assert moved(w=dict(W, **{name: W[name] * factor})) > 1e-4, name
    c = copy.deepcopy(BALELORN_A)
    c["layers"][0]["mlp"]["expert"]["limit"] = 0.5
    assert moved(c) > 1e-3
    assert moved(w=dict(W, **{"l0.mlp.table": (W["l0.mlp.table"] + 1) % 6})) > 1e-2
    assert moved(w=dict(W, **{"l1.mix.vmix": W["l1.mix.vmix"] + 5.0})) == 0.0       # the source's own number is never read
