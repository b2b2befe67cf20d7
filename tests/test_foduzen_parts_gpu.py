"""Each mechanism of the Foduzen decoder alone, as its kernels or its part, against the plain functions
(tests/plain_foduzen.py): the embedding with sinusoidal positions (far positions, odd widths); the sum of normed terms that
joins the stream; the activation with two numbers as rows and in the product kernels' epilogues at every number of tokens;
the short convolution over its ring; the recurrent unit's gates on both kinds of pipes, channels that forget at once beside
channels that keep everything; the recurrent unit, the gated attention (key and value heads of equal and of different sizes)
and the state-space recurrence as mixers, whole, in portions cut inside, at and around their chunks down to two tokens, token
by token, and in mixed steps on reused slots; one key whose score stands out just inside and just outside a window, at a page's
border and far back, on the tensor-core kernels too; the gated norm in groups."""
import pytest
import torch

import plain_foduzen as pf
from test_pilutar_parts_gpu import DEV, F64, TORCH, dev, ints, run_mixer, runs

pytestmark = pytest.mark.gpu
BF16 = torch.bfloat16


def bf(t):
    return t.to(BF16)


def close(got, want, tolerance, what=""):
    got, want = got.detach().cpu().to(F64), want.to(F64)
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    error = float((got - want).abs().max())
    assert error <= tolerance * max(1.0, float(want.abs().max())), f"{what}: {error:.3e}"


# ---- embedding, norms, activation ----

@pytest.mark.parametrize("hidden", [2, 5, 64, 257, 2048])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_embedding_with_sinusoidal_positions(hidden, dtype):
    from lia_rs_b200.kernels import ops
    g = torch.Generator().manual_seed(hidden)
    table = torch.randn(19, hidden, generator=g).to(TORCH[dtype])
    tokens, positions = [0, 18, 7, 7, 3], [0, 1, 2, 500, 30000]
    freq = (10000.0 ** (-2.0 * torch.arange((hidden + 1) // 2, dtype=F64) / hidden)).to(torch.float32)
    want = pf.embedding(torch.tensor(tokens), torch.tensor(positions), table, 3.5)
    out, copy = torch.empty(5, hidden, device=DEV), torch.empty(5, hidden, dtype=TORCH[dtype], device=DEV)
    ops.embedding_sinusoidal(ints(tokens), ints(positions), dev(table), dev(freq), out, 3.5, copy=copy)
    close(out[:4], want[:4], 4e-5, "positions up to 500")
    close(out[4:], want[4:], 3e-3, "position 30,000")           # a 32-bit angle of 30,000 is good to 2e-3
    assert torch.equal(copy, out.to(TORCH[dtype]))
    flag = torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.embedding_sinusoidal(ints([19]), ints([4]), dev(table), dev(freq), out[:1], 1.0, error_flag=flag)
    torch.cuda.synchronize()
    assert int(flag) == 1 and float(out[0].abs().max()) == 0.0


@pytest.mark.parametrize("hidden,rows", [(8, 3), (50, 5), (256, 4), (1028, 7), (2048, 2), (4096, 3), (8192, 2), (8196, 2)])
def test_terms_normed_into_the_stream(hidden, rows):
    from lia_rs_b200.kernels import ops
    g = torch.Generator().manual_seed(hidden)
    r = lambda *shape: torch.randn(*shape, generator=g)
    y, z, x, b, wy, wz, w = r(rows, hidden) * 4, r(rows, hidden), r(rows, hidden), r(hidden), r(hidden), r(hidden), r(hidden)
    d = lambda t: t.to(F64)
    both = 0.5 * pf.rms(d(y) + d(b), 1e-3) * d(wy) - 0.25 * pf.rms(d(z), 1e-5) * d(wz)
    cases = [([ops.NormTerm(dev(y), bias=dev(b), weight=dev(wy), scale=0.5, eps=1e-3),
               ops.NormTerm(dev(z), weight=dev(wz), scale=-0.25, eps=1e-5)], both),
             ([ops.NormTerm(dev(y))], d(y)), ([ops.NormTerm(dev(y), bias=dev(b), scale=2.0)], 2.0 * (d(y) + d(b))),
             ([ops.NormTerm(dev(y), bias=dev(b)), ops.NormTerm(dev(z), scale=3.0)], d(y) + d(b) + 3.0 * d(z))]
    for terms, total in cases:
        want = d(x) + pf.rms(total, 2e-5) * d(w)
        for dtype in (None, torch.float32, BF16):
            stream = dev(x.clone())
            copy = None if dtype is None else torch.empty(rows, hidden, dtype=dtype, device=DEV)
            ops.norm_terms_residual(terms, dev(w), stream, 2e-5, next_out=copy)
            close(stream, want, 2e-5)
            assert copy is None or torch.equal(copy, stream.to(dtype))


def test_a_single_number_as_norm_weight():
    from lia_rs_b200.parts import NORMS, Runtime
    g = torch.Generator().manual_seed(4)
    x = torch.randn(6, 40, generator=g)
    params = {"hidden": 40, "eps": 1e-4, "tensor": "", "single": True}
    cls = NORMS["rmsnorm"]
    assert [tuple(s.shape) for s in cls.tensor_specs(params, "n")] == [()]
    norm = cls(params, {"n": dev(bf(torch.tensor(-1.7)))}, "n", Runtime(DEV, torch.float32))
    out = torch.empty(6, 40, device=DEV)
    norm.forward(None, dev(x), out)
    close(out, pf.rms(x.to(F64), 1e-4) * float(bf(torch.tensor(-1.7))), 2e-6)
    assert norm.rms_record()[0].numel() == 40


@pytest.mark.parametrize("n", [1, 8, 16, 17, 40, 129, 520])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hidden,ff", [(64, 96), (128, 320), (50, 33), (512, 4096)])
def test_feed_forward_with_two_number_activation(n, dtype, hidden, ff):
    """Every product kernel that may serve the up product (few tokens, cluster, persistent, 32-bit pipes)."""
    from lia_rs_b200.cache import CacheManager
    from lia_rs_b200.engine import StepEntry, StepRuntime
    from lia_rs_b200.parts import FEED_FORWARDS, Runtime
    g = torch.Generator().manual_seed(hidden + ff)
    w = {"up": bf(torch.randn(ff, hidden, generator=g) * 2 / hidden ** 0.5), "down": bf(torch.randn(hidden, ff, generator=g) / ff ** 0.5),
         "act": bf(torch.tensor([0.7, -1.3]))}
    x = bf(torch.randn(n, hidden, generator=g))
    params = {"hidden": hidden, "intermediate": ff, "activation": "xielu", "names": {"up": "up", "down": "down", "act": "act"}}
    cache = CacheManager({}, {}, 64, 16, 4, 1024, TORCH[dtype], DEV)
    step = StepRuntime(cache, 100, 1024, DEV)
    slot = cache.admit()
    cache.ensure(slot, 0, n)
    ctx = step.begin([StepEntry(slot, [1] * n, 0, [])])
    part = FEED_FORWARDS["dense_act"](params, {k: dev(v) for k, v in w.items()}, "", Runtime(DEV, TORCH[dtype]))
    out = torch.zeros(n, hidden, device=DEV)
    part.forward(ctx, dev(x).to(TORCH[dtype]), out, 1.0)
    torch.cuda.synchronize()
    step.raise_device_errors()
    close(out, pf.dense_mlp(x.to(F64), w), 2e-5 if dtype == "float32" else 1.5e-2)


def test_activation_rows_around_zero_and_far_out():
    from lia_rs_b200.kernels import ops
    z = torch.cat([torch.linspace(-30, 30, 241), torch.tensor([0.0, 1e-6, -1e-6, 1e-3, -1e-3, -100.0])]).view(1, -1)
    p, q = torch.tensor(0.3, dtype=F64), torch.tensor(-2.0, dtype=F64)
    constants = (float(pf.softplus(p)), 0.5 + float(pf.softplus(q)))
    out = torch.empty_like(z, device=DEV)
    ops.activation_rows(dev(z), out, ops.ACT_XIELU, constants=constants)
    want = pf.xielu(z.to(F64), p, q)
    assert torch.allclose(out.cpu().to(F64), want, atol=1e-7, rtol=3e-6)


# ---- the short convolution over its ring ----

@pytest.mark.parametrize("channels,taps,act", [(8, 4, 1), (13, 3, 0), (64, 8, 1), (100, 1, 0), (516, 2, 1)])
def test_short_convolution_over_a_ring(channels, taps, act):
    """Portions of every size from one token on, two requests interleaved, the inputs of a run's end stored behind each step:
    every cut equals the convolution over the whole sequence."""
    from lia_rs_b200.kernels import ops
    g = torch.Generator().manual_seed(channels)
    T = 60
    x, b, ib = torch.randn(2, T, channels, generator=g), torch.randn(channels, generator=g), torch.randn(channels, generator=g)
    w = torch.randn(channels, taps, generator=g)
    want = [pf.causal_conv(x[r].to(F64) + ib.to(F64), w, b) for r in range(2)]
    if act:
        want = [pf.silu(v) for v in want]
    ring = torch.full((3, taps, channels), 7.0, device=DEV)             # what an earlier request left: never read before the start
    got = [[], []]
    at = [0, 0]
    for sizes in [(5, 1), (1, 1), (2, 9), (1, 0), (3, 2), (17, 1), (0, 30), (2, 1), (1, 1), (28, 14)]:
        plan = [(2 if r else 0, at[r], c) for r, c in enumerate(sizes) if c]
        positions, slots, *_ = runs(plan)
        rows = torch.cat([x[r, at[r]:at[r] + c] for r, c in enumerate(sizes)])
        wide = torch.zeros(rows.shape[0], channels + 4)
        wide[:, :channels] = rows
        wide = dev(wide)
        for dtype, store in ((torch.float32, True), (BF16, False)):
            out = torch.empty(rows.shape[0], channels, dtype=dtype, device=DEV)
            ops.ring_conv(wide, dev(ib), dev(w.t().contiguous()), dev(b), ring, positions, slots, out, act=act)
            if store:
                keep = out.cpu()
            else:
                close(out, keep, 1e-2)
        if taps > 1:
            ops.ring_store(wide, dev(ib), ring, positions, slots)
        first = 0
        for r, c in enumerate(sizes):
            got[r].append(keep[first:first + c])
            first += c
            at[r] += c
    for r in range(2):
        assert at[r] == T
        close(torch.cat(got[r]), want[r], 1e-5, f"request {r}")


# ---- the recurrent unit ----

@pytest.mark.parametrize("n", [1, 5, 33, 200])
@pytest.mark.parametrize("size,blocks", [(8, 3), (48, 5), (128, 1), (136, 2), (256, 2), (10, 5), (320, 1)])
def test_gates_on_both_kinds_of_pipes(size, blocks, n):
    from lia_rs_b200.kernels import ops
    g = torch.Generator().manual_seed(size + n)
    width = size * blocks
    u = bf(torch.randn(n, width, generator=g) * 2)
    wr, wi = (bf(torch.randn(blocks, size, size, generator=g) * 2 / size ** 0.5) for _ in range(2))
    bias = torch.randn(2, width, generator=g)
    lam = torch.linspace(-16, 9, width)                  # rates from 1e-6 (keeps everything) to 70 (forgets at once)
    rate = 8.0 * torch.nn.functional.softplus(lam)
    r = torch.sigmoid(pf.block_linear(u.to(F64), wr, bias[0].view(blocks, size)))
    i = torch.sigmoid(pf.block_linear(u.to(F64), wi, bias[1].view(blocks, size)))
    log_a = -rate.to(F64) * r
    want_a, want_b = torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * i * u.to(F64)
    slots = ints([0] * n)
    forms = []
    if ops.rglru_gates_tc_accepts(width, blocks):
        forms.append(lambda a, b: ops.rglru_gates_tc(dev(u), dev(wr), dev(wi), dev(bias), dev(rate), slots, a, b, blocks))
    both = torch.cat([wr.transpose(1, 2), wi.transpose(1, 2)], dim=2).contiguous()
    forms.append(lambda a, b: ops.rglru_gates(dev(u), dev(both), dev(bias), dev(rate), slots, a, b, blocks))
    forms.append(lambda a, b: ops.rglru_gates(dev(u.float()), dev(both.float()), dev(bias), dev(rate), slots, a, b, blocks))
    assert len(forms) == (3 if size % 8 == 0 else 2)
    for form in forms:
        a, b = torch.full((n, width), -5.0, device=DEV), torch.full((n, width), -5.0, device=DEV)
        form(a, b)
        assert float((a.cpu().to(F64) - want_a).abs().max()) <= 2e-6
        assert torch.allclose(b.cpu().to(F64), want_b, atol=1e-6, rtol=2e-5)      # relative: inflows of 1e-3 where a is close to one


def rglru_case(seed, hidden, width, blocks, taps, T):
    g = torch.Generator().manual_seed(seed)
    r = lambda *shape: torch.randn(*shape, generator=g)
    size = width // blocks
    w = {"y": bf(r(width, hidden) / hidden ** 0.5), "y.b": bf(r(width)), "x": bf(r(width, hidden) / hidden ** 0.5), "x.b": bf(r(width)),
         "conv": bf(r(width, taps)), "conv.b": bf(r(width)), "ra": bf(2 * r(blocks, size, size) / size ** 0.5),
         "ra.b": bf(r(blocks, size)), "ri": bf(2 * r(blocks, size, size) / size ** 0.5), "ri.b": bf(r(blocks, size)),
         "lam": bf(-9.0 + 13.0 * torch.rand(width, generator=g)), "o": bf(r(hidden, width) / width ** 0.5)}
    return bf(r(T, hidden)).to(F64), w


CUTS = [lambda T: [(0, T)], lambda T: [(0, 7), (7, 2), (9, 3), (12, 1), (13, 64), (77, T - 77)],
        lambda T: [(0, 31), (31, 2), (33, 32)] + [(t, 1) for t in range(65, T)], lambda T: [(t, 1) for t in range(T)]]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,blocks,taps", [(96, 3, 4), (40, 1, 2), (50, 5, 3), (64, 4, 1), (264, 3, 8), (512, 2, 4)])
def test_recurrent_unit(width, blocks, taps, dtype):
    hidden, T = 64, 300 if width == 512 else 110
    h, w = rglru_case(width, hidden, width, blocks, taps, T)
    want = pf.rglru(h, w)
    params = {"hidden": hidden, "width": width, "blocks": blocks, "taps": taps}
    for cut in CUTS[:3 if width == 512 else 4]:
        got = run_mixer("rglru", params, w, h, dtype, cut(T))
        close(got, want, 2e-5 if dtype == "float32" else 3e-2, f"{cut(T)[:2]}")


def test_the_recurrence_along_a_long_portion_and_mixed_runs():
    """The scan kernel alone: portions longer than what its warps take at once, several runs and single tokens in one step,
    slots in any order, channels that are not a multiple of 32; rows of nobody are left alone."""
    from lia_rs_b200.kernels import ops
    g = torch.Generator().manual_seed(6)
    width, taps = 70, 3
    plan = [(3, 11, 700), (0, 0, 1), (1, 40, 257), (2, 5, 2)]
    positions, slots, segments, n_segments, singles, _ = runs(plan)
    n = positions.numel()
    a = torch.rand(n, width, generator=g) ** 0.05
    a[:, ::7] = 1e-5
    b, wide = torch.randn(n, width, generator=g), torch.randn(n, 2 * width + 4, generator=g)
    yb, xb = torch.randn(width, generator=g), torch.randn(width, generator=g)
    state = torch.randn(5, taps * width + 2 + width, generator=g)
    device = dev(state.clone())
    ring, memory = device[:, :taps * width].view(5, taps, width), device[:, taps * width + 2:]
    out = torch.zeros(n, width, device=DEV)
    rows = dev(wide)
    ops.rglru_scan(dev(a), dev(b), rows[:, :width], rows[:, width:2 * width], dev(yb), dev(xb), ring, memory, segments, n_segments,
                   singles, positions, slots, out, taps)
    at = 0
    for slot, start, count in plan:
        S = state[slot, taps * width + 2:].to(F64)
        for t in range(at, at + count):
            S = a[t].to(F64) * S + b[t].to(F64)
            if t in (at, at + 1, at + count // 2, at + count - 1):
                want = S * pf.gelu_tanh(wide[t, :width].to(F64) + yb.to(F64))
                assert torch.allclose(out[t].cpu().to(F64), want, atol=2e-4, rtol=2e-5), (slot, t)
        assert torch.allclose(memory[slot].cpu().to(F64), S, atol=2e-4, rtol=2e-5)
        for k in range(min(taps, count)):
            p = start + count - 1 - k
            assert torch.allclose(ring[slot, p % taps].cpu(), wide[at + count - 1 - k, width:2 * width] + xb, atol=1e-6)
        at += count
    assert torch.equal(device[4].cpu(), state[4])


# ---- the gated attention ----

LEFT = [dict(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.25, mask={"size": 11}),
        dict(heads=3, kv_heads=3, dim=24, vdim=8, scale=0.2),
        dict(heads=8, kv_heads=1, dim=64, vdim=64, scale=0.125, mask={"size": 33}),
        dict(heads=4, kv_heads=4, dim=64, vdim=128, scale=0.125, mask={"size": 24}),
        dict(heads=16, kv_heads=2, dim=64, vdim=128, scale=0.1),
        dict(heads=8, kv_heads=2, dim=128, vdim=64, scale=0.09, mask={"size": 70}),
        dict(heads=24, kv_heads=2, dim=64, vdim=128, scale=0.125, mask={"size": 50}),    # 12 query heads a key head: no tcgen05 prompt kernel
        dict(heads=6, kv_heads=2, dim=32, vdim=64, scale=0.2, mask={"size": 40}),
        dict(heads=2, kv_heads=1, dim=64, vdim=32, scale=0.15, mask={"size": 200})]


def attention_weights(seed, hidden, m, sharp=2.0):
    g = torch.Generator().manual_seed(seed)
    r = lambda *shape: torch.randn(*shape, generator=g)
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    mat = lambda rows: bf(r(rows, hidden) / hidden ** 0.5)
    return {"q": mat(H * d), "k": mat(G * d), "v": mat(G * dv), "g": mat(H * dv), "o": bf(r(hidden, H * dv) / (H * dv) ** 0.5),
            "q.b": bf(0.3 * r(H * d)), "k.b": bf(0.3 * r(G * d)), "v.b": bf(0.3 * r(G * dv)), "o.b": bf(r(hidden)),
            "q.norm": bf(sharp * (1 + 0.2 * r(d))), "k.norm": bf(sharp * (1 + 0.2 * r(d)))}


def attention_params(hidden, m, eps):
    return {"hidden": hidden, "heads": m["heads"], "kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
            "scale": m["scale"], "window": m["mask"]["size"] if "mask" in m else None, "biases": True, "qk_norm": True,
            "norm_eps": eps, "gate": "sigmoid"}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", LEFT)
def test_gated_attention(m, dtype):
    hidden, T, eps = 72, 150, 1e-4
    w = attention_weights(m["heads"] + m["dim"], hidden, m)
    h = bf(torch.randn(T, hidden, generator=torch.Generator().manual_seed(3))).to(F64)
    want = pf.gated_attention(h, torch.arange(T), w, m, eps) - w["o.b"].to(F64)       # (the output's bias is the arrangement's)
    for cut in CUTS[:3]:
        got = run_mixer("sink_attention", attention_params(hidden, m, eps), w, h, dtype, cut(T))
        close(got, want, 2e-5 if dtype == "float32" else 4e-2, f"{cut(T)[:2]}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("page,window", [(16, 17), (8, 40), (4, 1), (16, 128)])
@pytest.mark.parametrize("d,dv", [(64, 128), (128, 64), (64, 64), (32, 64), (16, 8)])
def test_a_window_s_edge(d, dv, page, window, dtype):
    """One key's score stands out: the output is that key's value while the key is inside the window, also as its oldest one,
    and not when it is the first one outside; queries in a prompt portion and as single tokens; keys at a page's border, inside a
    page, at the sequence's start."""
    from lia_rs_b200.cache import CacheManager
    from lia_rs_b200.engine import StepEntry, StepRuntime
    from lia_rs_b200.parts.paged_attention import PagedAttention
    T = 200
    g = torch.Generator().manual_seed(d + page)
    k, v = bf(torch.randn(T, 1, d, generator=g)), bf(torch.randn(T, 1, dv, generator=g))
    targets = [t for t in (0, page - 1, page, 37, 59) if t + window < T]
    q = torch.zeros(T, 2, d)                                     # two query heads; each row asks for one target, or for nothing
    asks = {}
    for target in targets:
        for distance in (window - 1, window):
            asks.setdefault(target + distance, target)
    for t, target in asks.items():
        q[t, :] = 60.0 * k[target, 0].float() / float(k[target, 0].float().norm() ** 2)
    q = bf(q)
    scores = torch.einsum("ihd,jd->hij", q.to(F64), k[:, 0].to(F64))
    visible = pf.window_mask(torch.arange(T), window)
    p = torch.softmax(scores.masked_fill(~visible[None], float("-inf")), dim=-1)
    want = torch.einsum("hij,jv->ihv", p, v[:, 0].to(F64)).reshape(T, 2 * dv)
    for t, target in asks.items():
        assert (float(p[0, t, target]) > 0.9) if t - target == window - 1 else float(p[0, t, target]) == 0.0
    from lia_rs_b200.kernels import ops
    cache = CacheManager({0: _request(d, dv, window)}, {}, 64, page, 2, 1024, TORCH[dtype], DEV)
    step = StepRuntime(cache, 100, 512, DEV)
    paged = PagedAttention(TORCH[dtype], 2, 1, d, window, 1.0, v_head_dim=dv) if dtype == "bfloat16" and \
        PagedAttention.takes(d, dv, 2) else None
    for cut in ([(0, T)], [(0, 30), (30, 2), (32, 100), (132, 68)], [(0, window + 1)] + [(t, 1) for t in range(window + 1, T)]):
        slot = cache.admit()
        rows = []
        for start, count in cut:
            assert cache.ensure(slot, start, start + count)
            ctx = step.begin([StepEntry(slot, [1] * count, start, [])])
            kv = ctx.kv_view(0, True)
            for i in range(start, start + count):
                page_id = int(cache.kv_view(0, True).block_table[slot, i // page])
                kv.k_pages[page_id, i % page] = dev(k[i]).to(TORCH[dtype])
                kv.v_pages[page_id, i % page] = dev(v[i]).to(TORCH[dtype])
            torch.cuda.synchronize()
            qs = dev(q[start:start + count].reshape(count, 2 * d)).to(TORCH[dtype])
            out = torch.zeros(count, 2 * dv, dtype=TORCH[dtype], device=DEV)
            if paged is not None:
                paged.forward(ctx, qs, kv, out)
            else:
                ops.attention_general(qs, (2 * d, d), None, None, kv.k_pages, None, kv.v_pages, dv, dv, ctx.positions, ctx.slots,
                                      kv.block_table, out, (2 * dv, dv), count, 2, 1, window, 1.0)
            torch.cuda.synchronize()
            step.raise_device_errors()
            rows.append(out.cpu().to(F64))
        cache.release(slot)
        close(torch.cat(rows), want, 1e-5 if dtype == "float32" else 2e-2, f"cut {cut[:2]}")


def _request(d, dv, window):
    from lia_rs_b200.parts import KVCacheRequest
    return KVCacheRequest(1, d, window, v_head_dim=dv)


@pytest.mark.parametrize("window", [None, 300])
@pytest.mark.parametrize("d,dv,heads,kv_heads", [(64, 128, 8, 2), (128, 64, 4, 4), (32, 64, 12, 1), (64, 32, 6, 3), (64, 128, 24, 2)])
def test_unequal_head_sizes_with_keys_cut_into_ranges(d, dv, heads, kv_heads, window):
    """A token's keys cut into ranges that meet through scratch memory (by the last of its CTAs and by the merging kernel) and as
    clusters; a portion's keys cut into ranges of the prompt kernel where it takes the sizes."""
    from lia_rs_b200.kernels import ops
    g = torch.Generator().manual_seed(d + dv + heads)
    T, page = 700, 16
    pages = (T + page - 1) // page
    k, v = bf(torch.randn(pages * page, kv_heads, d, generator=g)), bf(torch.randn(pages * page, kv_heads, dv, generator=g))
    q = bf(torch.randn(T, heads, d, generator=g))
    order = torch.randperm(pages, generator=g)
    kp, vp = torch.empty(pages, page, kv_heads, d, dtype=BF16), torch.empty(pages, page, kv_heads, dv, dtype=BF16)
    kp[order], vp[order] = k.view(pages, page, kv_heads, d), v.view(pages, page, kv_heads, dv)
    kp, vp, table = dev(kp), dev(vp), ints(order.tolist()).view(1, pages)
    scale = d ** -0.5
    visible = pf.window_mask(torch.arange(T), window)
    want = torch.zeros(T, heads, dv, dtype=F64)
    for a in range(heads):
        scores = q[:, a].to(F64) @ k[:T, a // (heads // kv_heads)].to(F64).T * scale
        want[:, a] = torch.softmax(scores.masked_fill(~visible, float("-inf")), dim=-1) @ v[:T, a // (heads // kv_heads)].to(F64)
    want = want.reshape(T, heads * dv)
    positions, slots, qd = ints(range(T)), ints([0] * T), dev(q.reshape(T, heads * d))
    picked = [0, 63, 64, 299, 300, 301, 699]
    rows = ints(picked)
    groups = kv_heads * ((heads // kv_heads + 15) // 16)
    for splits in (1, 3, 11):
        for counted in (True, False):
            partial = torch.full((T * heads * splits * (dv + 1),), float("nan"), device=DEV) if splits > 1 else None
            counters = torch.zeros(len(picked) * groups, dtype=torch.int32, device=DEV) if counted else None
            out = torch.zeros(T, heads * dv, dtype=BF16, device=DEV)
            ops.attention_decode(qd, kp, vp, rows, positions, slots, table, out, partial, heads, kv_heads, d, window, scale, 0, splits,
                                 counters)
            close(out[picked], want[picked], 1.5e-2, f"{splits} ranges, counted {counted}")
            assert counters is None or int(counters.abs().max()) == 0
    fit = ops.attention_decode_cluster_splits(d, heads // kv_heads, len(picked) * groups, 8, dv)
    if fit > 1:
        out = torch.zeros(T, heads * dv, dtype=BF16, device=DEV)
        ops.attention_decode(qd, kp, vp, rows, positions, slots, table, out, None, heads, kv_heads, d, window, scale, 0, fit, None,
                             cluster=True)
        close(out[picked], want[picked], 1.5e-2, f"clusters of {fit}")
    per_tile = ops.attention_prefill_tc_tokens_per_tile(heads // kv_heads, d, dv)
    assert (per_tile > 0) == (d >= 64 and dv >= 64 and 128 % (heads // kv_heads) == 0)
    if per_tile:
        for splits in (1, 3):
            segments = ints([0, 0, 500, 500, 500, 200])
            tiles = -(-500 // per_tile) - (-200 // per_tile)
            partial = torch.full((ops.attention_prefill_tc_partial_floats(T, heads, dv, splits),), float("nan"), device=DEV) if splits > 1 else None
            out = torch.zeros(T, heads * dv, dtype=BF16, device=DEV)
            ops.attention_prefill_tc(qd, kp, vp, segments, 2, tiles, slots, table, out, heads, kv_heads, d, window, scale,
                                     splits=splits, partial=partial)
            close(out, want, 1.5e-2, f"portions, {splits} ranges")


# ---- the state-space recurrence ----

RIGHT = [dict(heads=4, vdim=12, state=20, groups=2, norm_groups=4, conv=3), dict(heads=3, vdim=8, state=6, groups=1, norm_groups=1, conv=5),
         dict(heads=1, vdim=32, state=32, groups=1, norm_groups=2, conv=4), dict(heads=8, vdim=6, state=10, groups=8, norm_groups=3, conv=8),
         dict(heads=4, vdim=64, state=64, groups=2, norm_groups=1, conv=4), dict(heads=2, vdim=64, state=128, groups=1, norm_groups=2, conv=4),
         dict(heads=6, vdim=32, state=16, groups=3, norm_groups=2, conv=1), dict(heads=2, vdim=128, state=48, groups=2, norm_groups=1, conv=2),
         dict(heads=2, vdim=200, state=256, groups=1, norm_groups=1, conv=4), dict(heads=2, vdim=40, state=24, groups=1, norm_groups=1, conv=4)]


def ssd_case(seed, hidden, m, T):
    g = torch.Generator().manual_seed(seed)
    r = lambda *shape: torch.randn(*shape, generator=g)
    inner, conv = m["heads"] * m["vdim"], m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
    w = {"in": bf(r(inner + conv + m["heads"], hidden) / hidden ** 0.5), "conv": bf(0.6 * r(conv, m["conv"])), "conv.b": bf(0.3 * r(conv)),
         "dt_bias": bf(-0.5 + r(m["heads"])), "A_log": bf(torch.linspace(-7, 3, m["heads"]) if m["heads"] > 1 else torch.tensor([-4.0])),
         "D": bf(r(m["heads"])), "norm": bf(1 + 0.3 * r(inner)), "o": bf(r(hidden, inner) / inner ** 0.5)}
    return bf(r(T, hidden)).to(F64), w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", RIGHT)
def test_state_space_recurrence(m, dtype):
    """Heads that forget within a token beside heads that keep hundreds of tokens."""
    hidden, T, eps = 64, 150, 1e-5
    h, w = ssd_case(m["heads"] + m["state"], hidden, m, T)
    want = pf.mamba2(h, w, m, eps)
    params = {"hidden": hidden, "heads": m["heads"], "size": m["vdim"], "state": m["state"], "groups": m["groups"],
              "norm_groups": m["norm_groups"], "taps": m["conv"], "norm_eps": eps}
    for cut in CUTS:
        got = run_mixer("state_space", params, w, h, dtype, cut(T))
        close(got, want, 3e-5 if dtype == "float32" else 3e-2, f"{cut(T)[:2]}")


@pytest.mark.parametrize("heads,P,N,G", [(4, 64, 64, 2), (2, 16, 16, 1), (6, 32, 48, 3), (3, 128, 128, 1), (2, 48, 96, 2),
                                          (1, 64, 256, 1), (2, 80, 16, 2), (8, 32, 112, 4)])
def test_state_space_portions_on_the_tensor_cores(heads, P, N, G):
    """bfloat16 x, B and C given, so that nothing but the kernels' own sums and powers differs from the plain recurrence: portions
    of 2 to 300 tokens in one step, from states in slots, heads that forget at once beside heads that keep everything; the same
    rows on the 32-bit pipes and, as single tokens, in place."""
    from lia_rs_b200.kernels import ops
    assert ops.ssd_tc_accepts(N, P)
    g = torch.Generator().manual_seed(heads * P + N)
    r = lambda *shape: torch.randn(*shape, generator=g)
    plan = [(2, 0, 129), (0, 7, 2), (3, 4, 300), (1, 9, 128), (4, 0, 33)]
    positions, slots, segments, n_segments, _, n = runs(plan)
    inner = heads * P
    xbc, wide = bf(r(n, inner + 2 * G * N)), r(n, heads + 3) * 2
    dt_bias, A_log, D = -1.0 + r(heads), torch.linspace(-8, 3, heads), r(heads)
    state = r(6, heads, N, P)
    arguments = [dev(dt_bias), dev(torch.exp(A_log)), dev(D)]
    results = []
    for rows in (dev(xbc), dev(xbc.float())):
        memory, y = dev(state.clone()), torch.zeros(n, inner, device=DEV)
        chunks = ops.ssd_chunks(n, n_segments, rows.dtype == BF16)
        scratch = torch.empty(ops.ssd_scratch_floats(chunks, heads, N, P), device=DEV)
        ops.ssd(rows, dev(wide)[:, 3:], *arguments, memory, segments, n_segments, chunks, slots, y, heads, G, N, P, scratch)
        results.append((y.cpu().to(F64), memory.cpu().to(F64)))
    at = 0
    for slot, start, count in plan:
        part = xbc[at:at + count].to(F64)
        want, last = pf.head_recurrence(part[:, :inner].reshape(count, heads, P), part[:, inner:inner + G * N].reshape(count, G, N),
                                        part[:, inner + G * N:].reshape(count, G, N),
                                        pf.softplus(wide[at:at + count, 3:].to(F64) + dt_bias.to(F64)), A_log, D, state[slot])
        for (y, memory), tolerance in zip(results, (6e-5, 2e-5)):
            assert float((y[at:at + count] - want.reshape(count, inner)).abs().max()) <= tolerance * max(1.0, float(want.abs().max()))
            assert float((memory[slot] - last).abs().max()) <= tolerance * max(1.0, float(last.abs().max()))
        if slot == 0:
            for rows in (dev(xbc), dev(xbc.float())):
                memory = dev(state.clone())
                for t in range(at, at + count):
                    y = torch.zeros(n, inner, device=DEV)
                    ops.ssd_single(dev(wide)[:, 3:], *arguments, memory, ints([t]), slots, y, heads, G, N, P, xbc=rows)
                    close(y[t], want[t - at].reshape(-1), 5e-6)
                close(memory[slot], last, 5e-6)
        at += count
    assert torch.equal(results[0][1][5].float(), state[5])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["rglru", "state_space"])
def test_mixed_runs_on_reused_slots(kind, dtype):
    """Portions beside single tokens of several requests in one step; a slot that is given back and taken again starts from
    zero; every request equals itself alone."""
    from lia_rs_b200.cache import CacheManager
    from lia_rs_b200.engine import StepEntry, StepRuntime
    from lia_rs_b200.parts import MIXERS, Runtime
    hidden, lengths = 64, [100, 45, 80, 70]
    if kind == "rglru":
        params = {"hidden": hidden, "width": 96, "blocks": 3, "taps": 4}
        h, w = rglru_case(9, hidden, 96, 3, 4, sum(lengths))
        plain = lambda rows: pf.rglru(rows, w)
    else:
        m = RIGHT[4]
        params = {"hidden": hidden, "heads": m["heads"], "size": m["vdim"], "state": m["state"], "groups": m["groups"],
                  "norm_groups": m["norm_groups"], "taps": m["conv"], "norm_eps": 1e-5}
        h, w = ssd_case(11, hidden, m, sum(lengths))
        plain = lambda rows: pf.mamba2(rows, w, m, 1e-5)
    inputs = list(h.split(lengths))
    cls = MIXERS[kind]
    cache = CacheManager({}, {0: cls.state_request(params)}, 32, 8, 3, 1024, TORCH[dtype], DEV)
    step = StepRuntime(cache, 100, 1024, DEV)
    part = cls(params, {k: v.to(DEV) for k, v in w.items()}, "", Runtime(DEV, TORCH[dtype]))
    slots, at, got = {}, [0] * 4, [[] for _ in lengths]
    plan = [{0: 33, 1: 1}, {0: 1, 1: 2, 2: 64}, {1: 42, 2: 1, 0: 1}, {0: 65, 2: 15, 3: 1}, {3: 2}, {3: 1}, {3: 66}]
    for batch in plan:
        entries = []
        for r, count in batch.items():
            if r not in slots:
                slots[r] = cache.admit()
            cache.ensure(slots[r], at[r], at[r] + count)
            entries.append(StepEntry(slots[r], [1] * count, at[r], []))
        ctx = step.begin(entries)
        rows = torch.cat([inputs[r][at[r]:at[r] + c] for r, c in batch.items()])
        out = torch.full((rows.shape[0], hidden), 5.0, device=DEV)
        part.forward(ctx, dev(rows).to(TORCH[dtype]), out, 1.0, state=ctx.state(0), store=True)
        torch.cuda.synchronize()
        step.raise_device_errors()
        first = 0
        for r, c in batch.items():
            got[r].append(out[first:first + c].cpu())
            first += c
            at[r] += c
            if at[r] == lengths[r]:
                cache.release(slots[r])                  # request 3 takes the slot of request 1
    for r, rows in enumerate(inputs):
        close(torch.cat(got[r]), plain(rows), 3e-5 if dtype == "float32" else 3e-2, f"request {r}")


@pytest.mark.parametrize("groups,size", [(1, 40), (3, 7), (8, 64), (2, 2048)])
def test_gated_norm_in_groups(groups, size):
    from lia_rs_b200.kernels import ops
    g = torch.Generator().manual_seed(size)
    y, wide, w = torch.randn(5, groups * size, generator=g) * 3, torch.randn(5, groups * size + 6, generator=g), torch.randn(groups * size, generator=g)
    want = pf.grouped_gated_norm(y.to(F64), wide[:, 2:2 + groups * size].to(F64), w, groups, 1e-4)
    for dtype, tolerance in ((torch.float32, 1e-5), (BF16, 1e-2)):
        out = torch.full((5, groups * size), 9.0, dtype=dtype, device=DEV)
        ops.gated_group_norm(dev(y), dev(wide)[:, 2:2 + groups * size], dev(w), ints([0, 1, -1, 0, 2]), out, groups, 1e-4)
        close(out[[0, 1, 3, 4]], want[[0, 1, 3, 4]], tolerance)
        assert float(out[2].float().min()) == 9.0
