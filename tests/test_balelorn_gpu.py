"""The engine's Balelorn model against the plain implementation: every mechanism alone, then whole models under every
way of cutting the work (whole prompts, a decoded tail, portions down to two tokens, mixed batches with pages and
slots used again, long decoding, generation through the scheduler), in 32-bit and in bfloat16, on configurations
that differ in every size, constant and in the order of layers."""
import random
from types import SimpleNamespace

import pytest
import torch

import plain_balelorn as pb
import replay_util as ru
from balelorn_configs import CONFIGS, make_folder
from test_safepel_gpu import CUTS, MixerHarness, load_part, random_tensors, rel, run_in_cuts

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = {"float32": (torch.float32, 5e-5), "bfloat16": (torch.bfloat16, 3e-2)}
# beside the cuts of the other mixers' tests: portions of two requests in one step long enough for the prompt kernels
ALL_CUTS = dict(CUTS, **{"large portions": [(70, 30), (50, 7), (30, 0)]})


def inputs(hidden, lens, seed, dt):
    g = torch.Generator().manual_seed(seed)
    return [torch.randn(n, hidden, generator=g).to(dt).float() for n in lens]


def floats(w):
    return {k: v.float() if v.is_floating_point() else v.long() for k, v in w.items()}


# ------------------------------------------------------------------ attention alone
def att_spec(hidden, H, G, D, V, scale, chunk=None, rot=None, mix=None, prefix="m."):
    from ferrox_b200.parts.specs import AttentionSpec, ScaledRotarySpec, ValueMixSpec

    return AttentionSpec(
        hidden=hidden, n_heads=H, n_kv_heads=G, head_dim=D, value_dim=V, qkv_bias=False, window=None, prefix=prefix,
        position=ScaledRotarySpec(*rot) if rot else None, softmax_scale=scale, output_gate="g", chunk=chunk, sink="sink",
        tensor_names=(("q", "q"), ("k", "k"), ("v", "v"), ("o", "o")),
        value_mix=None if mix is None else ValueMixSpec("vmix", source=mix == "source"))


def att_mixer(H, G, D, V, scale, chunk=None, rot=None):
    m = dict(heads=H, kv_heads=G, dim=D, vdim=V, scale=scale)
    if chunk:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return m


class TwoLayers(MixerHarness):
    """The source of the values and a layer that mixes with them, on the same rows; the second one's output."""

    def __init__(self, first, part, rt, hidden, **kw):
        from ferrox_b200.cache.manager import CacheManager

        super().__init__(part, rt, hidden, **kw)
        self.first = first
        self.mgr = CacheManager([part.cache_spec(), first.cache_spec()], page_size=self.mgr.page_size,
                                n_pages=kw.get("n_pages", 64), max_slots=3, max_positions=self.mgr.max_positions, device=DEV,
                                dtype=rt.dtype)
        inner, harness = part, self

        class Both:
            def forward_into(self, x, out, batch, cache, accumulate=False):
                harness.first.forward_into(x, torch.empty_like(out), batch, harness.mgr.layer_cache(1), accumulate=False)
                inner.forward_into(x, out, batch, cache, accumulate=accumulate)
        self.part = Both()


SHAPES = [  # heads, kv heads, dim, vdim, chunk, (rot dims, base), page
    (4, 2, 32, 48, 24, (16, 500.0), 8), (3, 3, 20, 12, 13, (6, 1000.0), 4), (6, 1, 12, 36, None, (12, 33.0), 16),
    (8, 2, 64, 64, 64, (32, 20000.0), 64), (4, 1, 128, 128, 100, (128, 250000.0), 64), (6, 3, 96, 40, 70, (48, 500.0), 64),
    (2, 2, 24, 24, 1, None, 64), (40, 1, 64, 64, 33, (2, 10.0), 64), (4, 2, 128, 56, 37, (64, 10000.0), 128),
    (70, 1, 16, 16, 50, (16, 99.0), 16)]


@pytest.mark.parametrize("cut", list(ALL_CUTS))
@pytest.mark.parametrize("mix", [None, "source", "mixed"])
@pytest.mark.parametrize("H,G,D,V,chunk,rot,page", SHAPES)
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_attention_alone(dtype, H, G, D, V, chunk, rot, page, mix, cut):
    """Rotation, chunks, sink, mixing of values and gate under every cut, two requests side by side; then the slots and
    pages are used again."""
    if mix is not None and cut == "portions" and dtype == "float32":
        pytest.skip("(the other cuts cover it)")
    dt, tol = DTYPES[dtype]
    hidden = 64
    scale = round(0.5 / D ** 0.5, 4)
    spec = att_spec(hidden, H, G, D, V, scale, chunk, rot, mix)
    w = random_tensors(spec, seed=H + D, std=0.25)
    w["m.sink"] = (torch.randn(H, generator=torch.Generator().manual_seed(V)) * 1.5 + 1.0).to(torch.bfloat16)
    m = att_mixer(H, G, D, V, scale, chunk, rot)
    xs = inputs(hidden, (150, 37), 3, dt)
    wf = floats(w)
    kw = dict(page_size=page, n_pages=256 // page + 8)
    if mix == "mixed":
        spec1 = att_spec(hidden, H, G, D, V, scale, chunk, rot, "source", prefix="f.")
        w1 = random_tensors(spec1, seed=7 * H + D, std=0.25)
        first_of = lambda x: pb.attention(m, floats(w1), "f.", x, None)[1]
        want = [pb.attention(m, wf, "m.", x, first_of(x))[0] for x in xs]
        assert rel(pb.attention(m, wf, "m.", xs[0], None)[0], want[0]) > 0.02       # the mixing shows
        first, _ = load_part(spec1, w1, dt)
        part, rt = load_part(spec, w, dt)
        h = TwoLayers(first, part, rt, hidden, **kw)
    else:
        want = [pb.attention(m, wf, "m.", x, None)[0] for x in xs]
        part, rt = load_part(spec, w, dt)
        h = MixerHarness(part, rt, hidden, **kw)
    got = run_in_cuts(h, xs, ALL_CUTS[cut])
    for a, b in zip(got, want):
        assert rel(a, b) < tol
    got = run_in_cuts(h, xs[::-1], [c[::-1] for c in ALL_CUTS[cut]])
    for a, b in zip(got, want[::-1]):
        assert rel(a, b) < tol
    h.mgr.check_invariants()


@pytest.mark.parametrize("D,V,page", [(32, 48, 8), (64, 64, 64), (128, 128, 64), (128, 40, 64)])
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_keys_at_a_chunks_and_a_pages_edges(dtype, D, V, page):
    """The first and the last key of every chunk, and the keys at page borders, are made to win the softmax of every
    query that may see them; queries in the next chunk may not.  In a prompt, in portions and decoded one by one.  The
    plain implementation with chunks one position longer or shorter gives something else, so the edge shows."""
    dt, tol = DTYPES[dtype]
    hidden, H, G, n, chunk = 64, 4, 2, 330, 70
    g = torch.Generator().manual_seed(2)
    spec = att_spec(hidden, H, G, D, V, 1.0, chunk, None)
    w = random_tensors(spec, seed=D, std=0.25)
    x = torch.randn(n, hidden, generator=g) * 0.3
    # one direction of the input is the queries' and keys' common first element; loud rows carry it
    u = torch.zeros(hidden)
    u[0] = 1.0
    for name, heads in (("q", H), ("k", G)):
        wt = w["m." + name].float() * 0.05
        wt.view(heads, D, hidden)[:, 0] = u * 1.5
        w["m." + name] = wt.to(torch.bfloat16)
    x[:, 0] = 1.0
    loud = [p for c in range(0, n, chunk) for p in (c, c + chunk - 1) if p < n] + [63, 64, 127, 128, 191, 192]
    x[loud, 0] = torch.linspace(3.0, 6.0, len(loud))[torch.randperm(len(loud), generator=g)]
    x = x.to(dt).float()
    m, wf = att_mixer(H, G, D, V, 1.0, chunk), floats(w)
    want = pb.attention(m, wf, "m.", x, None)[0]
    for other in (chunk - 1, chunk + 1):
        off = pb.attention(dict(m, mask={"size": other}), wf, "m.", x, None)[0]
        assert float((off - want).abs().max(dim=1).values[chunk:].max() / want.abs().max()) > 0.1
    part, rt = load_part(spec, w, dt)
    for cuts in ([(n,)], [(9,), (2,), (58,), (2,), (69,), (130,), (60,)], [(69,)] + [(1,)] * 261, [(140,)] + [(1,)] * 150 + [(40,)]):
        got = run_in_cuts(MixerHarness(part, rt, hidden, page_size=page, n_pages=512 // page + 8), [x], cuts)
        assert rel(got[0], want) < tol


@pytest.mark.parametrize("shift", [0.0, -40.0, 25.0])
def test_sinks_from_nothing_to_everything(shift):
    """A sink far below the scores changes nothing, one far above them takes (nearly) all the weight: no overflow, in
    every kernel."""
    hidden, H, G, D = 64, 4, 1, 64
    for dtype, (dt, tol) in DTYPES.items():
        spec = att_spec(hidden, H, G, D, D, 0.1, 90, (32, 1000.0))
        w = random_tensors(spec, seed=5, std=0.25)
        w["m.sink"] = (w["m.sink"].float() + shift).to(torch.bfloat16)
        part, rt = load_part(spec, w, dt)
        xs = inputs(hidden, (150, 37), 4, dt)
        m = att_mixer(H, G, D, D, 0.1, 90, (32, 1000.0))
        want = [pb.attention(m, floats(w), "m.", x, None)[0] for x in xs]
        for cut in ("whole", "one by one", "large portions"):
            got = run_in_cuts(MixerHarness(part, rt, hidden, page_size=64, n_pages=16), xs, ALL_CUTS[cut])
            for a, b in zip(got, want):
                assert torch.isfinite(a).all() and rel(a, b) < tol


def plain_attention(q, k, v, pos, chunk, window, scale, sinks, gate):
    """One query row [H, D] against keys [n, G, D] and values [n, G, V]; everything 64-bit."""
    H, G = q.shape[0], k.shape[1]
    lo = 0
    if chunk:
        lo = pos // chunk * chunk
    if window:
        lo = max(lo, pos - window + 1)
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (k[lo:pos + 1, g].double() @ q[h].double()) * scale
        e = torch.exp(s - s.max())
        den = e.sum() + (torch.exp(sinks[h].double() - s.max()) if sinks is not None else 0.0)
        out.append((e / den) @ v[lo:pos + 1, g].double())
    o = torch.stack(out)
    return o * torch.sigmoid(gate.double()).view_as(o) if gate is not None else o


def paged(keys, values, page_size, seed):
    """Keys and values of one request in shuffled pages (one unused page between): pages and a block table row."""
    n, G, D = keys.shape
    V = values.shape[2]
    n_pages = -(-n // page_size)
    order = torch.randperm(n_pages + 2, generator=torch.Generator().manual_seed(seed))[:n_pages]
    kp, vp = torch.zeros(n_pages + 2, G, page_size, D), torch.zeros(n_pages + 2, G, page_size, V)
    for i in range(n_pages):
        part = slice(i * page_size, min(n, (i + 1) * page_size))
        kp[order[i], :, :part.stop - part.start] = keys[part].transpose(0, 1)
        vp[order[i], :, :part.stop - part.start] = values[part].transpose(0, 1)
    return kp, vp, order.to(torch.int32)[None]


@pytest.mark.parametrize("run_blocks", [0, 2])
@pytest.mark.parametrize("D,V,chunk,window,sink,gate", [
    (128, 128, 400, None, True, True), (64, 64, None, None, True, False), (128, 48, 640, None, True, True),
    (96, 128, 300, None, False, True), (40, 72, None, 200, True, True), (8, 8, 1000, None, True, True),
    (64, 104, 256, 100, False, False)])
def test_prompt_kernel_with_runs_of_key_blocks(D, V, chunk, window, sink, gate, run_blocks):
    """The tcgen05 prompt kernel and its merge: key and value widths of their own, chunks, sinks, gate; a portion behind
    a long prefix, tiles cut into runs of key blocks or whole."""
    from ferrox_b200.kernels import ops

    g = torch.Generator().manual_seed(D + V)
    H, G, page, start, n = 4, 2, 64, 900, 340
    bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    q, k, v = bf(n, H * D), bf(start + n, G, D), bf(start + n, G, V)
    gates, sinks = (bf(n, H * V) if gate else None), (torch.randn(H, generator=g) * 2 if sink else None)
    kp, vp, table = paged(k.float(), v.float(), page, 3)
    dev = lambda t, dt=None: None if t is None else (t.to(DEV) if dt is None else t.to(DEV).to(dt)).contiguous()
    items, merges, parts = ops.prefill_tc_plan([(n, start)], window, H, run_blocks=run_blocks, chunk=chunk)
    assert (parts > 0) == (run_blocks > 0)
    out = torch.full((n, H * V), float("nan"), dtype=torch.bfloat16, device=DEV)
    part_o = torch.full((max(1, parts), H, 256, ops.prefill_value_width(V)), float("nan"), device=DEV)
    part_ml = torch.full((max(1, parts), H, 256, 2), float("nan"), device=DEV)
    scale = 1.3 / D ** 0.5
    ops.prefill_attention_tc(dev(q), dev(kp, torch.bfloat16), dev(vp, torch.bfloat16), dev(table), page,
                             torch.from_numpy(items).to(DEV), torch.zeros(1, dtype=torch.int32, device=DEV), out, H, G, D,
                             window, scale, merges=torch.from_numpy(merges).to(DEV) if parts else None, part_o=part_o,
                             part_ml=part_ml, value_dim=V, chunk=chunk, sinks=dev(sinks), gate=dev(gates))
    assert torch.isfinite(out).all()
    for i in list(range(0, n, 23)) + [n - 1, 255, 256]:
        want = plain_attention(q[i].float().view(H, D), k.float(), v.float(), start + i, chunk, window, scale, sinks,
                               gates[i].float() if gate else None)
        assert rel(out[i].view(H, V), want) < 2e-2, i


@pytest.mark.parametrize("n_splits", [1, 3, 7])
@pytest.mark.parametrize("merged_inside", [True, False])
@pytest.mark.parametrize("D,chunk,window,sink,gate", [(128, 400, None, True, True), (64, 70, None, True, False),
                                                      (128, None, 300, False, True), (64, 1000, 200, True, True)])
def test_decode_kernel_with_runs_of_keys(D, chunk, window, sink, gate, merged_inside, n_splits):
    """The decode kernel that streams pages by TMA: chunks, sinks and gate with one run of keys, with runs that the last
    block merges, and with runs that the second kernel merges."""
    from ferrox_b200.kernels import ops

    g = torch.Generator().manual_seed(D + n_splits)
    H, G, page, n = 8, 2, 64, 1000
    bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    k, v = bf(n, G, D), bf(n, G, D)
    positions = [0, 63, 64, 399, 400, 401, 777, 999]
    T = len(positions)
    q, gates = bf(T, H * D), (bf(T, H * D) if gate else None)
    sinks = torch.randn(H, generator=g) * 2 if sink else None
    kp, vp, table = paged(k.float(), v.float(), page, 4)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    dev = lambda t: None if t is None else t.to(DEV).contiguous()
    out = torch.full((T, H * D), float("nan"), dtype=torch.bfloat16, device=DEV)
    acc = torch.empty(T, H, n_splits, D, device=DEV)
    ml = torch.empty(T, H, n_splits, 2, device=DEV)
    counters = torch.zeros(1024, dtype=torch.int32, device=DEV) if merged_inside else None
    scale, gates_d, sinks_d = 1.3 / D ** 0.5, dev(gates), dev(sinks)
    ops.decode_attention(dev(q), dev(kp).to(torch.bfloat16), dev(vp).to(torch.bfloat16), dev(table), page, i32(positions),
                         i32([0] * T), i32([0]), out, H, G, D, window, scale, 0, n_splits, acc, ml, counters=counters,
                         extras=ops.DecodeExtras.of(chunk, sinks_d, gates_d))
    torch.cuda.synchronize()
    for i, p in enumerate(positions):
        want = plain_attention(q[i].float().view(H, D), k.float(), v.float(), p, chunk, window, scale, sinks,
                               gates[i].float() if gate else None)
        assert rel(out[i].view(H, D), want) < 2e-2, p
    assert counters is None or int(counters.abs().sum()) == 0


def test_a_layer_without_the_source_before_it_is_refused():
    spec = att_spec(64, 2, 1, 16, 16, 0.2, None, None, "mixed")
    part, rt = load_part(spec, random_tensors(spec, seed=1), torch.float32)
    with pytest.raises(RuntimeError, match="values"):
        run_in_cuts(MixerHarness(part, rt, 64), [torch.randn(5, 64)], [(5,)])


# ------------------------------------------------------------------ feed-forwards, norms, embedding alone
def step_batch(tokens):
    from ferrox_b200.engine.batch import StepEntry, flatten
    from ferrox_b200.kernels import ops

    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    return flatten([StepEntry(0, list(tokens), start=0)], torch.device(DEV), status, ops.stream_ptr())


def table_spec(hidden, E, top, I, limit, vocab, prefix="f."):
    from ferrox_b200.parts.specs import MoeSpec

    return MoeSpec(hidden=hidden, n_experts=E, top_k=top, expert_intermediate=I, shared_intermediate=0, norm_topk_prob=False,
                   shared_gate=False, prefix=prefix, activation=("clamped_swish", limit, 1.702),
                   tensor_names=("", "e{e}.{part}", ""), table="table", vocab=vocab)


@pytest.mark.parametrize("E,top,I", [(6, 2, 32), (3, 3, 24), (5, 1, 48), (8, 3, 64), (1, 1, 8), (70, 4, 32)])
@pytest.mark.parametrize("tokens", [1, 5, 40, 64, 300, 1500])
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_experts_chosen_by_a_table_alone(dtype, tokens, E, top, I):
    """Two layers whose tables one launch serves, added to a stream, written into a buffer, and with the norm behind
    them, the addition and the next norm in the kernel that adds a token's rows up."""
    from ferrox_b200.parts.base import build_part
    from ferrox_b200.parts.specs import NormSpec
    from ferrox_b200.weights import loader as wl

    dt, tol = DTYPES[dtype]
    hidden, vocab, limit = 64, 37, 1.2
    specs = [table_spec(hidden, E, top, I, limit, vocab, p) for p in ("f.", "g.")]
    ws = [random_tensors(s, seed=tokens + top + i, std=0.3) for i, s in enumerate(specs)]
    _, rt = load_part(specs[0], ws[0], dt)
    rt.groups.clear()
    parts = []
    for s, w in zip(specs, ws):
        p = build_part(s)
        p.load(wl.from_dict(w, p.tensor_decls(), DEV, dt), rt)
        parts.append(p)
    x = inputs(hidden, [tokens], 5, dt)[0]
    rng = random.Random(tokens)
    toks = [rng.randrange(vocab) for _ in range(tokens)]
    f = {"router": {"experts": E, "top": top}, "expert": {"ff": I, "limit": limit}}
    batch = step_batch(toks)
    norms = [load_part(NormSpec(hidden, 1e-5, "", name=n), {n: (1 + 0.2 * torch.randn(hidden)).to(torch.bfloat16)}, dt)[0]
             for n in ("a", "b")]
    xd = x.to(DEV).to(dt)
    for part, w, p in zip(parts, ws, ("f.", "g.")):
        want = pb.table_experts(f, floats(w), p, x, toks)
        h = torch.ones(tokens, hidden, device=DEV)
        part.forward_add(xd, h, batch)
        assert rel(h - 1, want) < tol
        out = torch.full((tokens, hidden), float("nan"), device=DEV)
        part.forward_into(xd, out, batch, accumulate=False)
        assert rel(out, want) < tol
        h0 = torch.randn(tokens, hidden, generator=torch.Generator().manual_seed(8))
        h = h0.to(DEV)
        nxt = part.forward_post(xd, h, batch, norms[0], norms[1])
        new = h0 + pb.rms_norm(want, norms[0].weight.float().cpu(), 1e-5)
        assert rel(h, new) < tol and rel(nxt, pb.rms_norm(new, norms[1].weight.float().cpu(), 1e-5)) < tol
        h = h0.to(DEV)
        assert part.forward_post(xd, h, batch, norms[0]) is None and rel(h, new) < tol
    assert len([k for k in batch.shared]) == 1 and len(rt.groups[("expert tables", vocab, top, E)]) == 2


def test_tables_that_do_not_fit_are_refused():
    from ferrox_b200 import WeightsError

    spec = table_spec(64, 4, 2, 32, 1.0, 9)
    good = random_tensors(spec, seed=1)
    for row in ([1, 1], [0, 4], [-1, 2]):
        w = dict(good)
        w["f.table"] = good["f.table"].clone()
        w["f.table"][3] = torch.tensor(row, dtype=torch.int32)
        with pytest.raises(WeightsError, match="different experts"):
            load_part(spec, w, torch.float32)


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_gelu_gated_feed_forward_alone(dtype):
    from ferrox_b200.kernels import ops
    from ferrox_b200.parts.specs import DenseMlpSpec

    dt, tol = DTYPES[dtype]
    for hidden, ff in ((96, 160), (72, 50), (256, 448)):
        spec = DenseMlpSpec(hidden=hidden, intermediate=ff, prefix="f.", tensor_names=("gate", "up", "down"), activation="gelu_tanh")
        w = random_tensors(spec, std=0.2)
        part, _ = load_part(spec, w, dt)
        for T in (1, 3, 20, 70, 300, 2304):     # the decode-sized and the prompt-sized kernels, pairs of SMs
            x = torch.randn(T, hidden, generator=torch.Generator().manual_seed(T)).to(dt)
            out = torch.full((T, hidden), float("nan"), device=DEV)
            part.forward_into(x.to(DEV), out, SimpleNamespace(status=None, stream=ops.stream_ptr()), accumulate=False)
            assert rel(out, pb.dense(None, floats(w), "f.", x.float())) < tol
    # the gate's arithmetic where it is far from the origin: zeros and the identity, no overflow
    z = torch.tensor([-300.0, -30.0, -9.0, -1.0, 0.0, 1e-4, 1.0, 9.0, 30.0, 300.0])
    gu = torch.cat([z, torch.ones(10)])[None].to(DEV).to(dt).contiguous()
    out = torch.empty(1, 10, dtype=dt, device=DEV)
    ops.silu_mul(gu, out, activation="gelu_tanh")
    assert rel(out[0], pb.gelu_tanh(z.to(dt).float())) < 1e-2 and torch.isfinite(out).all()


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_norm_of_a_sublayers_output_added_and_the_next_norm(dtype):
    from ferrox_b200.kernels import ops

    dt = DTYPES[dtype][0]
    g = torch.Generator().manual_seed(1)
    for rows, hidden in ((1, 64), (7, 72), (300, 200), (5, 2048), (3, 5000), (400, 4096), (2, 10000), (3, 16384), (3, 4099)):
        h, y = torch.randn(rows, hidden, generator=g), torch.randn(rows, hidden, generator=g) * 3
        w, wn = (1 + 0.2 * torch.randn(hidden, generator=g)), (1 + 0.2 * torch.randn(hidden, generator=g)).to(torch.bfloat16)
        hd, out = h.to(DEV), torch.empty(rows, hidden, dtype=dt, device=DEV)
        assert ops.rmsnorm_residual_ok(hd)
        got = ops.rmsnorm_residual(hd, y.to(DEV), w.to(DEV), 3e-6, then=(wn.to(DEV), 1e-5, out))
        new = h + pb.rms_norm(y, w, 3e-6)
        assert got is out and rel(hd, new) < 2e-6
        assert rel(out, pb.rms_norm(new, wn.float(), 1e-5)) < (1e-5 if dt == torch.float32 else 1e-2)
        hd = h.to(DEV)
        assert ops.rmsnorm_residual(hd, y.to(DEV), w.to(DEV), 3e-6) is None and rel(hd, new) < 2e-6


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_normed_embedding_and_a_norm_with_a_scale(dtype):
    from ferrox_b200.kernels import ops
    from ferrox_b200.parts.specs import NormSpec

    dt = DTYPES[dtype][0]
    g = torch.Generator().manual_seed(3)
    table, w = torch.randn(50, 72, generator=g).to(dt), (1 + 0.3 * torch.randn(72, generator=g)).to(torch.bfloat16)
    ids = torch.tensor([0, 49, 7, 7], dtype=torch.int32)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.empty(4, 72, device=DEV)
    ops.embed_norm(table.to(DEV), ids.to(DEV), w.to(DEV), 1e-5, out, status=status)
    assert rel(out, pb.rms_norm(table.float()[ids.long()], w.float(), 1e-5)) < 1e-6 and int(status) == 0
    ops.embed_norm(table.to(DEV), torch.tensor([50, 1], dtype=torch.int32, device=DEV), w.to(DEV), 1e-5, out[:2], status=status)
    assert int(status) == 1 and float(out[0].abs().max()) == 0.0            # an id outside the vocabulary raises the status
    ls = torch.randn(72, generator=g).to(torch.bfloat16)
    part, _ = load_part(NormSpec(72, 1e-5, "", name="n", scale_name="s"), {"n": w, "s": ls}, dt)
    x = torch.randn(6, 72, generator=g)
    want = pb.rms_norm(x, w.float(), 1e-5) * ls.float()
    assert rel(part.forward(x.to(DEV)), want) < (1e-6 if dt == torch.float32 else 1e-2)
    xd = x.to(DEV)
    assert rel(part.forward_in_place(xd), want) < 1e-6 and rel(xd, want) < 1e-6


# ------------------------------------------------------------------ whole models
def prompts_for(name, n=5, hi=150, seed=0):
    cfg = CONFIGS[name][0]
    rng = random.Random(seed)
    lens = [1, 2, hi] + [rng.randint(3, hi) for _ in range(max(0, n - 3))]
    return {f"r{i}": [rng.randrange(cfg["vocab"]) for _ in range(L)] for i, L in enumerate(lens)}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("balelorn_models")
    return {name: make_folder(tmp, name) for name in CONFIGS}


def position_errors(got, want):
    return (got - want).abs().amax(dim=-1) / want.abs().max()


def rounding_alone(cfg, w, tokens, want):
    """Per position: how far the plain implementation's logits move when everything that may be computed in bfloat16
    is rounded to it."""
    with pb.rounded_to(torch.bfloat16):
        return position_errors(pb.forward(cfg, w, tokens), want)


@pytest.fixture(scope="module")
def expected(folders):
    out = {}
    for name in CONFIGS:
        cfg, w = CONFIGS[name][0], pb.load_weights(folders[name])
        want = {rid: pb.forward(cfg, w, t) for rid, t in prompts_for(name).items()}
        out[name] = (cfg, w, want, {rid: rounding_alone(cfg, w, t, want[rid]) for rid, t in prompts_for(name).items()})
    return out


def engine(folder, dtype, **kw):
    from ferrox_b200 import Engine

    kw.setdefault("page_size", 64 if folder.endswith("_C") else 8)     # C: the page size of serving
    kw.setdefault("n_pages", 64)
    kw.setdefault("max_slots", 4)
    return Engine.from_folder(folder, dtype=dtype, **kw)


def compare(got, want, tol, what, noise=None):
    """32-bit: every position within ``tol``.  bfloat16 (``noise``: what rounding alone does to the plain
    implementation at every position): every position within four times the largest of that, and the median within
    twice the median, plus a thousandth."""
    errs = []
    for rid in want:
        assert got[rid].shape == want[rid].shape, (what, rid)
        assert torch.isfinite(got[rid]).all(), (what, rid)
        e = position_errors(got[rid], want[rid])
        if noise is None:
            assert float(e.max()) < tol, (what, rid, float(e.max()), int(e.argmax()))
        errs.append(e)
    if noise is not None:
        e, n = torch.cat(errs), torch.cat([noise[rid] for rid in want])
        assert float(e.max()) <= 4 * float(n.max()), (what, float(e.max()), float(n.max()))
        assert float(e.median()) <= 2 * float(n.median()) + 1e-3, (what, float(e.median()), float(n.median()))


RUNS = {
    "whole": lambda eng, p: ru.run_whole(eng, p),
    "decoded tail": lambda eng, p: ru.run_tail_decode(eng, p, tail=50),
    "portions": lambda eng, p: ru.run_portions(eng, p),
    "decoding together": lambda eng, p: ru.run_decode_together(eng, p, tail=9),
    "mixed": lambda eng, p: ru.run_mixed(eng, p, seed=3, max_live=3),
    "mixed, large portions": lambda eng, p: ru.run_mixed(eng, p, seed=6, max_live=4, max_portion=60),
}


@pytest.mark.parametrize("run", list(RUNS))
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_model_under_every_cut(folders, expected, dtype, name, run):
    _, tol = DTYPES[dtype]
    eng = engine(folders[name], dtype)
    got = RUNS[run](eng, prompts_for(name))
    compare(got, expected[name][2], tol, f"{name} {dtype} {run}", expected[name][3] if dtype == "bfloat16" else None)
    eng.cache.check_invariants()
    assert all(n == eng.cache.groups[k].pool.n_pages for k, n in eng.cache.free_pages().items())   # all given back


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_cuts_agree_with_each_other_to_rounding(folders, name):
    eng = engine(folders[name], "float32")
    p = prompts_for(name)
    whole, mixed = ru.run_whole(eng, p), ru.run_mixed(eng, p, seed=5, max_live=4)
    for rid in p:
        assert float((whole[rid] - mixed[rid]).abs().max() / whole[rid].abs().max()) < 2e-5


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_residual_stream_after_every_layer(folders, expected, name):
    from ferrox_b200.engine.batch import StepEntry

    cfg, w = expected[name][:2]
    toks = prompts_for(name)["r3"]
    want_logits, after = pb.forward(cfg, w, toks, return_layers=True)
    eng = engine(folders[name], "float32")
    seen = []
    for i, block in enumerate(eng.model.layers):
        inner = block.forward

        def spy(h, batch, cache, _inner=inner, _i=i, **kw):
            out = _inner(h, batch, cache, **kw)
            seen.append((_i, h.detach().clone().cpu()))
            return out
        block.forward = spy
    slot = eng.open_request()
    got = eng.step([StepEntry(slot, toks, want=list(range(len(toks))))]).cpu()
    assert [i for i, _ in seen] == list(range(len(cfg["layers"])))
    for n, (_, h) in enumerate(seen):
        assert rel(h, after[n]) < 2e-5, n
    assert rel(got, want_logits) < 5e-5


@pytest.mark.parametrize("name", ["A", "C"])
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_long_decoding(folders, dtype, name):
    """A few tokens of prompt, then hundreds decoded one by one, across many chunks and pages; the pool holds few pages,
    so that those of the chunks left behind are used again."""
    _, tol = DTYPES[dtype]
    cfg, w = CONFIGS[name][0], pb.load_weights(folders[name])
    rng = random.Random(9)
    n = 303 if name == "A" else 420
    toks = [rng.randrange(cfg["vocab"]) for _ in range(n)]
    want = pb.forward(cfg, w, toks)
    eng = engine(folders[name], dtype, n_pages=8 if name == "A" else 4, max_slots=2)      # 64 and 256 positions
    c = ru.Collector(eng)
    c.step({"x": toks[:3]})
    for t in toks[3:]:
        c.step({"x": [t]})
    compare({"x": c.stacked("x")}, {"x": want}, tol, "long decoding",
            {"x": rounding_alone(cfg, w, toks, want)} if dtype == "bfloat16" else None)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_greedy_generation_through_the_scheduler(folders, name):
    cfg, w = CONFIGS[name][0], pb.load_weights(folders[name])
    rng = random.Random(4)
    prompts = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (5, 1, 23)]
    want = [pb.greedy(cfg, w, p, 12) for p in prompts]
    eng = engine(folders[name], "float32")
    assert eng.graphs is not None            # every part of the model can be captured: decode steps replay graphs
    got = eng.generate(prompts, max_new_tokens=12, max_batch_tokens=16)     # prompts go in portions
    assert got == want
    again = eng.generate(prompts[::-1], max_new_tokens=12)                  # slots and pages used again
    assert again == want[::-1]
    bf = engine(folders[name], "bfloat16").generate(prompts, max_new_tokens=12)
    assert all(len(g) == 12 for g in bf)
    for p, g in zip(prompts, bf):
        logits = pb.forward(cfg, w, (p + g)[:-1])
        for i, tok in enumerate(g):
            row = logits[len(p) - 1 + i]
            assert float(row.max() - row[tok]) <= 2 * 6e-2 * float(logits.abs().max())


def test_trace_replay_and_command_line_with_a_balelorn_folder(folders, tmp_path):
    import json
    import os
    import subprocess
    import sys

    import numpy as np

    cfg, w = CONFIGS["B"][0], pb.load_weights(folders["B"])
    toks = [3, 90, 7, 7, 45, 21, 9, 81]
    want = pb.forward(cfg, w, toks)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": toks[:5], "want": [0, 4]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": toks[5:6], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": toks[6:], "want": [1]}, {"id": "b", "tokens": toks[:2], "want": [1]}],
         "end": ["a", "b"]},
    ]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders["B"], "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    s0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1))
    s2 = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4").reshape(2, -1))
    assert rel(s0, want[[0, 4]]) < 5e-5 and rel(s2, want[[7, 1]]) < 5e-5
    nxt = pb.greedy(cfg, w, toks[:4], 2)
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "ferrox"), "-m", folders["B"], "--tokens", "3,90,7,7",
                        "-n", "2", "--temp", "0", "--dtype", "float32", "--ignore-eos", "--repeat-penalty", "1.0"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(t) for t in r.stdout.split()] == nxt


def test_preemption_decoding_ahead_and_sampling(folders):
    """A request that is preempted gives its pages and slot back and is recomputed; greedy decode steps are replayed
    graphs issued one ahead of the host; sampled ones depend on the seed alone."""
    cfg, w = CONFIGS["B"][0], pb.load_weights(folders["B"])
    prompts = [[i + 1, i + 3, i + 7, 90, 4, 8, 15, 16] for i in range(4)]
    want = [pb.greedy(cfg, w, p, 20) for p in prompts]
    small = engine(folders["B"], "float32", page_size=4, n_pages=14, max_slots=4)     # 4 x 28 positions do not fit 56
    outs, stats = small.generate(prompts, max_new_tokens=20, return_stats=True)
    assert stats["preemptions"] >= 1 and outs == want
    small.cache.check_invariants()
    roomy = engine(folders["B"], "float32", n_pages=64)
    outs, stats = roomy.generate(prompts, max_new_tokens=20, return_stats=True)
    assert outs == want and stats["ahead_steps"] >= 8 and stats["preemptions"] == 0
    sampled = [roomy.generate(prompts, max_new_tokens=10, temperature=0.8, top_k=20, seed=s) for s in (1, 1, 2)]
    assert sampled[0] == sampled[1] and sampled[0] != sampled[2]
