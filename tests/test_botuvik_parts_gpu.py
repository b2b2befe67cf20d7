"""Each mechanism of the Botuvik decoder alone, as its kernels or its part, against the plain functions
(tests/plain_botuvik.py): interleaved rotation with the weightless norm behind it; attention with a learned sink a head and a
cap on the scores on every kernel that takes them (key and value heads of equal and unequal size, cut key ranges, groups of
query heads), with one key made to stand out far back, at a page's border and in place of the sink; the matrix memory whole,
in portions cut inside, at and around its chunks down to two tokens, token by token, in mixed steps on reused slots, on the
32-bit pipes and on the tensor cores, heads cut into pieces and shared by several CTAs, with gates that forget at once beside
gates that keep everything and with sums that must cancel; the router (sigmoid scores, groups judged by their two largest,
groups of one, ties) and the whole mixture with an ungated shared expert; the stream's step ahead of a pass."""
import pytest
import torch

import plain_botuvik as pb

pytestmark = pytest.mark.gpu
F64 = torch.float64
DEV = "cuda:0"
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
bf = lambda t: t.to(torch.bfloat16)


def dev(t, dtype=None):
    return t.to("cuda", dtype=dtype) if dtype else t.to("cuda")


def ints(values):
    return torch.tensor(list(values), dtype=torch.int32, device="cuda")


def off_by(got, want, dtype):
    """32-bit: the largest error.  bfloat16: the largest row's root-mean-square error, or a third of the largest error (a head's
    norm raises the rounding of a row whose sums cancel)."""
    error = (got - want).abs()
    return float(error.max()) if dtype == "float32" else max(float((error ** 2).mean(dim=-1).sqrt().max()), float(error.max()) / 3.0)


class PartRunner:
    """A mixer part alone over a cache manager and step runtime of its own: `step([(request, count)])` runs the next tokens of
    the named requests as one batch; a request's rows of `h` are consumed in order."""

    def __init__(self, kind, params, weights, dtype, page_size=8, slots=4, tokens=2048):
        from lia_rs_b200.cache import CacheManager
        from lia_rs_b200.engine import StepRuntime
        from lia_rs_b200.parts import MIXERS, Runtime
        cls = MIXERS[kind]
        self.dtype = TORCH[dtype]
        cache_request, state_request = cls.cache_request(params), cls.state_request(params)
        self.has_cache, self.has_state = cache_request is not None, state_request is not None
        self.cache = CacheManager({0: cache_request} if cache_request else {}, {0: state_request} if state_request else {}, tokens,
                                  slots, page_size, tokens, self.dtype, DEV)
        self.runtime = StepRuntime(self.cache, 1000, tokens, DEV)
        self.part = cls(params, {"L." + k: v.to(DEV) for k, v in weights.items()}, "L.", Runtime(DEV, self.dtype))
        self.live = {}

    def step(self, entries, rows):
        """rows: {request: [T, hidden]}; returns {request: what the part adds to a zero residual} for this step."""
        from lia_rs_b200.engine import StepEntry
        batch, inputs = [], []
        for name, count in entries:
            if name not in self.live:
                self.live[name] = [self.cache.admit(), 0]
            slot, at = self.live[name]
            assert self.cache.ensure(slot, at, at + count)
            batch.append(StepEntry(slot, [1] * count, at, []))
            inputs.append(rows[name][at:at + count])
            self.live[name][1] = at + count
        ctx = self.runtime.begin(batch)
        x = torch.cat(inputs).to(DEV).to(self.dtype)
        if x.shape[0] < ctx.n_tokens:                    # rows of nobody
            x = torch.cat([x, torch.zeros(ctx.n_tokens - x.shape[0], x.shape[1], dtype=self.dtype, device=DEV)])
        # (a step lists its single tokens and portions in the order of the entries)
        residual = torch.zeros(x.shape[0], x.shape[1], device=DEV)
        self.part.forward(ctx, x, residual, 1.0, kv=ctx.kv_view(0, True) if self.has_cache else None,
                          state=ctx.state(0) if self.has_state else None)
        torch.cuda.synchronize()
        self.runtime.raise_device_errors()
        out, at = {}, 0
        for name, count in entries:
            out[name] = residual[at:at + count].cpu().to(F64)
            at += count
        return out

    def end(self, name):
        self.cache.release(self.live.pop(name)[0])


def run_alone(kind, params, weights, h, dtype, sizes, page_size=8):
    runner = PartRunner(kind, params, weights, dtype, page_size)
    return torch.cat([runner.step([("r", n)], {"r": h})["r"] for n in sizes])


def cuts(T):
    yield [T]
    sizes, at, pattern = [], 0, [2, 3, 1, 2, 31, 1, 33, 2, 64]
    while at < T:
        n = min(pattern[len(sizes) % len(pattern)], T - at)
        sizes.append(n)
        at += n
    yield sizes
    yield [T // 2] + [1] * (T - T // 2)


# ---- attention ----

def attention_weights(seed, hidden, m, sink_at=1.0):
    g = torch.Generator().manual_seed(seed)
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    mat = lambda rows, cols: bf(torch.randn(rows, cols, generator=g) / cols ** 0.5)
    return {"q": mat(H * d, hidden), "k": mat(G * d, hidden), "v": mat(G * dv, hidden), "o": mat(hidden, H * dv),
            "q.b": bf(0.5 * torch.randn(H * d, generator=g)), "k.b": bf(0.5 * torch.randn(G * d, generator=g)),
            "v.b": bf(0.5 * torch.randn(G * dv, generator=g)), "sink": bf(sink_at + 2.0 * torch.randn(H, generator=g))}


def attention_params(hidden, m, eps):
    return {"hidden": hidden, "heads": m["heads"], "kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
            "scale": m["scale"], "softcap": m.get("softcap"), "rot": m.get("rot"), "rot_pairs": True, "biases": "qkv",
            "qk_norm": "behind", "norm_eps": eps, "sink": "learned"}


def _m(heads, kv_heads, dim, vdim, scale, softcap=None, rot=None):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, softcap=softcap,
                rot=None if rot is None else {"base": rot[0], "dims": rot[1]})


ATTENTION = [_m(4, 2, 20, 12, 0.3, 5.0, (1000.0, 12)), _m(3, 3, 24, 8, 0.4), _m(5, 1, 80, 96, 0.15, 30.0, (1e6, 80)),
             _m(8, 1, 64, 64, 0.3, 20.0, (1e5, 64)), _m(4, 4, 128, 128, 0.2, 50.0, (5e5, 64)), _m(4, 2, 64, 128, 0.25, 9.0, (1e4, 2)),
             _m(2, 1, 128, 64, 0.2, 15.0, (1e4, 128)), _m(4, 2, 64, 64, 0.3, None, (1e4, 64)),
             # three query heads a key head: portions go to the kernel for every size, single tokens to the split-key kernel
             _m(6, 2, 64, 64, 0.25, 8.0, (1e4, 32)), _m(6, 2, 64, 64, 0.25, None, (1e4, 32)),
             _m(32, 1, 32, 32, 0.4, 15.0, (1e4, 32)), _m(4, 2, 32, 64, 0.4, 10.0, (1e4, 16)), _m(4, 1, 64, 32, 0.3, 6.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", ATTENTION)
def test_attention_with_sinks_and_a_cap(m, dtype):
    hidden, T, eps = 72, 90, 1e-5
    w = attention_weights(m["heads"] + m["dim"], hidden, m)
    h = bf(torch.randn(T, hidden, generator=torch.Generator().manual_seed(1))).to(F64)
    want = pb.attention(h, torch.arange(T), w, m, eps)
    without = pb.attention(h, torch.arange(T), {**w, "sink": torch.full((m["heads"],), -50.0)}, m, eps)
    tolerance = (2e-5 if dtype == "float32" else 4e-2) * max(1.0, float(want.abs().max()))
    assert float((want - without).abs().max()) > 4 * tolerance               # a sink that is left out would show
    for sizes in cuts(T):
        got = run_alone("sink_attention", attention_params(hidden, m, eps), w, h, dtype, sizes)
        assert float((got - want).abs().max()) <= tolerance, sizes[:3]


@pytest.mark.parametrize("dtype,d,dv", [("float32", 24, 16), ("bfloat16", 64, 64), ("bfloat16", 128, 128), ("bfloat16", 64, 128)])
def test_long_contexts_cut_into_ranges(dtype, d, dv):
    """1,500 keys: single tokens whose keys the split-key kernel cuts (clusters, and scratch memory where many rows decode), and
    short late portions whose keys the prompt kernel cuts; the sink joins once, where the ranges meet."""
    m = _m(8, 2, d, dv, 0.3, 20.0, (1e5, d))
    hidden, T, eps = 64, 1500, 1e-5
    w = attention_weights(d, hidden, m, sink_at=5.0)
    h = bf(torch.randn(T, hidden, generator=torch.Generator().manual_seed(2))).to(F64)
    want = pb.attention(h, torch.arange(T), w, m, eps)
    without = pb.attention(h[1200:], torch.arange(1200, T), w, m, eps)         # (a rule of thumb for "far keys matter")
    tolerance = (3e-5 if dtype == "float32" else 4e-2) * max(1.0, float(want.abs().max()))
    assert float((want[1200:] - without).abs().max()) > tolerance
    for sizes in ([T], [1400] + [1] * 40 + [60], [1024, 300, 16, 2, 100, 58]):
        got = run_alone("sink_attention", attention_params(hidden, m, eps), w, h, dtype, sizes, page_size=16)
        assert float((got - want).abs().max()) <= tolerance, sizes[:3]


@pytest.mark.parametrize("softcap", [None, 6.0])
@pytest.mark.parametrize("path", ["general", "decode", "prefill"])
@pytest.mark.parametrize("target", [0, 15, 16, 37, 300])
def test_one_key_stands_out(target, path, softcap):
    """One query asks for exactly one key (its score alone is large): the output is nearly that key's value, times what the sink
    leaves of it.  The key is the first of all, the last of a page, the first of one, inside one, and the query's own."""
    from lia_rs_b200.kernels import ops
    g = torch.Generator().manual_seed(target)
    T, d, page, H = 301, 64, 16, 2
    dtype = torch.float32 if path == "general" else torch.bfloat16
    k, v = bf(torch.randn(T, 1, d, generator=g)), bf(torch.randn(T, 1, d, generator=g))
    q = torch.zeros(T, H, d)
    for h in range(H):
        q[T - 1, h] = 9.0 * k[target, 0].float() / float(k[target, 0].float().norm()) ** 2
    q = bf(q)
    sinks = torch.tensor([8.0, -3.0])
    want = pb.attend(q.to(F64), k.to(F64), v.to(F64), 1.0, softcap, sinks)[T - 1].reshape(-1)
    pages = (T + page - 1) // page
    fill = lambda x: dev(torch.cat([x, torch.zeros(pages * page - T, 1, d)]).view(pages, page, 1, d), dtype).contiguous()
    kp, vp, table = fill(k), fill(v), ints(range(pages)).view(1, pages)
    out = torch.zeros(T, H * d, dtype=dtype, device="cuda")
    qd, positions, slots = dev(q.reshape(T, H * d), dtype), ints(range(T)), ints([0] * T)
    common = dict(softcap=softcap, sinks=dev(sinks))
    if path == "general":
        ops.attention_general(qd, (H * d, d), None, None, kp, None, vp, d, d, positions, slots, table, out, (H * d, d), T, H, 1, None,
                              1.0, rows=ints([T - 1]), **common)
    elif path == "decode":
        ops.attention_decode(qd, kp, vp, ints([T - 1]), positions, slots, table, out, None, H, 1, d, None, 1.0, 0, 1, **common)
    else:
        per = ops.attention_prefill_tc_tokens_per_tile(H, d)
        ops.attention_prefill_tc(qd, kp, vp, ints([0, 0, T]), 1, (T + per - 1) // per, slots, table, out, H, 1, d, None, 1.0, **common)
    torch.cuda.synchronize()
    tolerance = 1e-5 if path == "general" else 2e-2
    assert float((out[T - 1].cpu().to(F64) - want).abs().max()) <= tolerance * max(1.0, float(want.abs().max()))
    value = v[target, 0].to(F64)
    share = float((want[d:] @ value) / (value @ value))
    assert share > (0.2 if softcap else 0.8)              # (the head with the small sink)
    assert float((want[:d] @ value) / (value @ value)) < share - 0.15


def test_rotation_in_pairs_and_the_norm_behind_it():
    """What the pages and the queries hold, element by element: pairs (2i, 2i+1), positions far from zero, the norm over the whole
    head with an eps that matters for a tiny one."""
    from lia_rs_b200.kernels import ops
    g = torch.Generator().manual_seed(4)
    nq, nkv, d, dv, dims, T, eps, page = 3, 1, 20, 8, 12, 6, 1e-3, 4
    rows = torch.randn(T, (nq + nkv) * d + nkv * dv, generator=g)
    rows[2] *= 1e-3                                       # a head of the size of eps
    bias = torch.randn(rows.shape[1], generator=g) * 0.1
    positions = torch.tensor([0, 1, 2, 1000, 65535, 7])
    freq = torch.tensor([1e4 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float32)
    q_out = torch.zeros(T, nq * d, device="cuda")
    pages = 65536 // page
    kp, vp = torch.zeros(pages, page, nkv, d, device="cuda"), torch.zeros(pages, page, nkv, dv, device="cuda")
    table = ints(range(pages)).view(1, pages)
    ops.qkv_prepare(dev(rows), dev(bias), None, None, eps, dev(freq), dims, 0, 0.0, None, ints(positions), ints([0] * T), table, q_out, kp,
                    vp, nq, nkv, d, dv, pairs=True, norm_behind=True)
    both = (rows + bias).to(F64)
    heads = pb.rms(pb.rotate_interleaved(both[:, :(nq + nkv) * d].view(T, nq + nkv, d), positions, 1e4, dims), eps)
    near = positions < 5000                               # (32-bit angles at 65,535 are good to about 1e-3)
    assert torch.allclose(q_out.cpu().to(F64).view(T, nq, d)[near], heads[near, :nq], atol=2e-4)
    keys = kp.view(-1, nkv, d)[positions.to("cuda")].cpu().to(F64)
    assert torch.allclose(keys[near], heads[near, nq:], atol=2e-4)
    assert torch.allclose(keys, heads[:, nq:], atol=2e-2)
    values = vp.view(-1, nkv * dv)[positions.to("cuda")].cpu().to(F64)
    assert torch.allclose(values, both[:, (nq + nkv) * d:], atol=1e-6)


# ---- the matrix memory ----

def memory_weights(seed, hidden, H, d, dv, forget=4.0, spread=2.5):
    g = torch.Generator().manual_seed(seed)
    mat = lambda rows, cols, s=1.0: bf(torch.randn(rows, cols, generator=g) * s / cols ** 0.5)
    return {"q": mat(H * d, hidden), "k": mat(H * d, hidden), "v": mat(H * dv, hidden), "g": mat(H * dv, hidden),
            "i": mat(H, hidden, 2.0), "f": mat(H, hidden), "i.b": bf(-1.0 + 2.0 * torch.randn(H, generator=g)),
            "f.b": bf(forget + spread * torch.randn(H, generator=g)), "norm": bf(1 + 0.3 * torch.randn(H * dv, generator=g)),
            "o": mat(hidden, H * dv)}


MEMORY = [(1, 6, 5, 8.0), (3, 10, 14, 15.0), (2, 33, 65, 4.0), (4, 16, 16, 12.0), (2, 64, 128, 15.0), (3, 48, 80, 10.0),
          (2, 32, 160, 15.0), (1, 128, 256, 15.0), (1, 256, 512, 15.0), (2, 80, 400, 9.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,d,dv,cap", MEMORY)
def test_matrix_memory(H, d, dv, cap, dtype):
    hidden, T, eps = 72, 270, 1e-5
    m = {"heads": H, "dim": d, "vdim": dv, "gate_cap": cap}
    w = memory_weights(d + dv, hidden, H, d, dv)
    h = bf(torch.randn(T, hidden, generator=torch.Generator().manual_seed(5))).to(F64)
    want, _ = pb.mlstm(h, w, m, eps)
    params = {"hidden": hidden, "heads": H, "head_dim": d, "v_head_dim": dv, "gate_cap": cap, "norm_eps": eps}
    tolerance = (1e-4 if dtype == "float32" else 5e-2) * max(1.0, float(want.abs().max()))
    for sizes in list(cuts(T)) + [[128, 127, 15], [32, 31, 33, 129, 45]]:
        got = run_alone("mlstm", params, w, h, dtype, sizes)
        assert off_by(got, want, dtype) <= tolerance, sizes[:3]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,d,dv", [(2, 10, 14), (2, 64, 128), (1, 64, 192)])
def test_matrix_memories_of_several_requests_on_reused_slots(H, d, dv, dtype):
    """Four slots, six requests: portions beside single tokens, three portions at once, slots whose memory, sum of keys and
    maximum another request has left."""
    hidden, eps = 48, 1e-5
    m = {"heads": H, "dim": d, "vdim": dv, "gate_cap": 12.0}
    w = memory_weights(d, hidden, H, d, dv)
    g = torch.Generator().manual_seed(6)
    lengths = {"a": 200, "b": 9, "c": 150, "d": 40, "e": 61, "f": 300}
    rows = {r: bf(torch.randn(n, hidden, generator=g)).to(F64) for r, n in lengths.items()}
    params = {"hidden": hidden, "heads": H, "head_dim": d, "v_head_dim": dv, "gate_cap": 12.0, "norm_eps": eps}
    runner = PartRunner("mlstm", params, w, dtype)
    got = {r: [] for r in lengths}
    plan = [[("a", 129), ("b", 2)], [("b", 1), ("a", 1), ("c", 5)], [("a", 2), ("b", 6), ("c", 130), ("d", 38)], [("e", 33), ("a", 1), ("d", 1)],
            [("c", 1), ("d", 1), ("e", 1), ("a", 1)], [("a", 66), ("c", 14)], [("f", 257), ("e", 27)], [("f", 1)], [("f", 42)]]
    for entries in plan:
        for name, out in runner.step(entries, rows).items():
            got[name].append(out)
        for name in [r for r, (_, at) in runner.live.items() if at == lengths[r]]:
            runner.end(name)
    for name, parts in got.items():
        want, _ = pb.mlstm(rows[name], w, m, eps)
        tolerance = (1e-4 if dtype == "float32" else 5e-2) * max(1.0, float(want.abs().max()))
        assert torch.cat(parts).shape == want.shape and off_by(torch.cat(parts), want, dtype) <= tolerance, name


@pytest.mark.parametrize("tensor_cores", [False, True])
@pytest.mark.parametrize("forget,what", [(-30.0, "forgets at once"), (0.0, "halves"), (9.0, "keeps thousands"), (None, "changes")])
def test_memory_kernels_with_extreme_gates(forget, what, tensor_cores):
    """The kernels from given q, k, v and gates against the recurrence: forget gates at both ends of the cap, where F of a chunk
    runs to more than a thousand while the exponents that matter are of order one, and input gates at both ends, where the
    divisor is once the sum of the keys and once exp(-m); the state after the last token too."""
    from lia_rs_b200.kernels import ops
    H, d, dv, T, cap, eps = 2, 32, 48, 400, 13.0, 1e-6
    g = torch.Generator().manual_seed(8)
    q, k, v = (bf(torch.randn(T, H, n, generator=g)) for n in (d, d, dv))
    gate = torch.randn(T, H * dv, generator=g)
    zi = 6.0 * torch.randn(T, H, generator=g)
    zf = torch.full((T, H), forget) if forget is not None else 20.0 * torch.randn(T, H, generator=g)
    i_bias, f_bias = torch.tensor([1.0, -8.0]), torch.tensor([0.5, 0.0])
    weight = 1 + 0.2 * torch.randn(H * dv, generator=g)
    squash = lambda z, b: cap * torch.tanh((z + b).to(F64) / cap)
    o, (S, n, m) = pb.mlstm_recurrence(q.to(F64) * d ** -0.5, k.to(F64), v.to(F64), squash(zi, i_bias),
                                       torch.nn.functional.logsigmoid(squash(zf, f_bias)))
    want = pb.rms(o, eps).reshape(T, -1) * weight.to(F64) * torch.sigmoid(gate.to(F64))
    qkv = torch.cat([t.reshape(T, -1) for t in (q, k, v)], dim=1)
    gates = dev(torch.cat([gate, zi, zf], dim=1))
    words = H * (d * dv + d + 1)
    for sizes in ([T], [130, 2, 1, 31, 1, 129, 106]):
        state = torch.zeros(3, (words + 3) // 4 * 4, device="cuda")
        outs, at = [], 0
        for count in sizes:
            rows = dev(qkv[at:at + count], torch.bfloat16 if tensor_cores else torch.float32).contiguous()
            out = torch.zeros(count, H * dv, dtype=torch.bfloat16 if tensor_cores else torch.float32, device="cuda")
            shared = (rows, gates[at:at + count], dev(i_bias), dev(f_bias), cap, state)
            if count == 1:
                ops.mlstm_single(*shared, ints([0]), ints([1]), dev(weight), eps, out, H, d, dv, wanted_ctas=0)
            else:
                chunks = ops.mlstm_chunks(count, 1, tensor_cores)
                scratch = torch.zeros(ops.mlstm_scratch_floats(chunks, H, d, dv), device="cuda")
                ops.mlstm(*shared, ints([0, at, count]), 1, chunks, ints([1] * count), dev(weight), eps, out, H, d, dv, scratch)
            outs.append(out.cpu().to(F64))
            at += count
        got = torch.cat(outs)
        scale = max(1.0, float(want.abs().max()))
        assert float((got - want).abs().max()) <= (2e-2 if tensor_cores else 2e-4) * scale, (what, sizes[:2])
        assert float(state[0].abs().max()) == 0 and float(state[2].abs().max()) == 0
        mine = state[1].cpu().to(F64)
        # (the state is exact up to 32-bit sums on both paths; m is a number of order one however long the sequence)
        assert torch.allclose(mine[words - H:words], m, atol=2e-4)
        assert torch.allclose(mine[:H * d * dv].view(H, d, dv), S, atol=3e-4 * max(1.0, float(S.abs().max())))
        assert torch.allclose(mine[H * d * dv:words - H].view(H, d), n, atol=3e-4 * max(1.0, float(n.abs().max())))


@pytest.mark.parametrize("share", [1, 2, 4, 8])
@pytest.mark.parametrize("qkv_dtype", [torch.float32, torch.bfloat16])
def test_single_tokens_by_several_ctas_a_head(share, qkv_dtype):
    """A head's value columns shared by 1, 2, 4 and 8 CTAs: the same outputs and the same state, and rows of nobody are skipped."""
    from lia_rs_b200.kernels import ops
    H, d, dv, n, cap, eps = 2, 40, 256, 3, 10.0, 1e-5
    g = torch.Generator().manual_seed(9)
    words = H * (d * dv + d + 1)
    start = torch.randn(5, (words + 3) // 4 * 4, generator=g)
    qkv, gates = torch.randn(n, H * (2 * d + dv), generator=g), torch.randn(n, H * (dv + 2), generator=g)
    qkv = bf(qkv).float()
    i_bias, f_bias, weight = torch.randn(H, generator=g), 2 + torch.randn(H, generator=g), 1 + 0.2 * torch.randn(H * dv, generator=g)
    state, out = dev(start.clone()), torch.full((n, H * dv), 7.0, device="cuda")
    slots = [3, -1, 0]
    ops.mlstm_single(dev(qkv, qkv_dtype), dev(gates), dev(i_bias), dev(f_bias), cap, state, ints(range(n)), ints(slots), dev(weight), eps,
                     out, H, d, dv, wanted_ctas=n * H * share)
    torch.cuda.synchronize()
    assert torch.equal(out[1].cpu(), torch.full((H * dv,), 7.0))
    for t, slot in ((0, 3), (2, 0)):
        row, mem = qkv[t].to(F64), start[slot].to(F64)
        part = lambda a, b, size: row[a:b].view(1, H, size)
        before = (mem[:H * d * dv].view(H, d, dv), mem[H * d * dv:words - H].view(H, d), mem[words - H:words])
        i = cap * torch.tanh((gates[t, H * dv:H * dv + H] + i_bias).to(F64) / cap)
        f = torch.nn.functional.logsigmoid(cap * torch.tanh((gates[t, H * dv + H:] + f_bias).to(F64) / cap))
        o, (S, nn, m) = pb.mlstm_recurrence(part(0, H * d, d) * d ** -0.5, part(H * d, 2 * H * d, d), part(2 * H * d, H * (2 * d + dv), dv),
                                            i[None], f[None], before)
        want = pb.rms(o[0], eps).reshape(-1) * weight.to(F64) * torch.sigmoid(gates[t, :H * dv].to(F64))
        assert torch.allclose(out[t].cpu().to(F64), want, atol=2e-5, rtol=2e-5)
        mine = state[slot].cpu().to(F64)
        assert torch.allclose(mine[:words], torch.cat([S.reshape(-1), nn.reshape(-1), m]), atol=2e-5, rtol=2e-5)
    for slot in (1, 2, 4):
        assert torch.equal(state[slot].cpu(), start[slot])


# ---- router, mixture, the stream's step ----

@pytest.mark.parametrize("experts,top,groups", [(10, 3, (5, 4)), (6, 2, (3, 2)), (4, 1, (4, 2)), (12, 5, (2, 1)), (7, 7, None), (1, 1, None),
                                                (64, 8, (8, 4)), (9, 3, (1, 1))])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_router(experts, top, groups, dtype):
    from lia_rs_b200.kernels import ops
    g = torch.Generator().manual_seed(experts * 10 + top)
    n, hidden = 200, 72
    h = bf(torch.randn(n, hidden, generator=g))
    router = torch.randn(experts, hidden, generator=g) * 2.0 / hidden ** 0.5
    spec = {"experts": experts, "top": top, **({"groups": {"count": groups[0], "keep": groups[1]}} if groups else {})}
    chosen, weights = pb.route(h.to(F64), {"router": router}, spec)
    s = torch.sigmoid(h.to(F64) @ router.to(F64).T)
    ids, w = torch.zeros(n, top, dtype=torch.int32, device="cuda"), torch.zeros(n, top, device="cuda")
    ops.moe_route(dev(h, TORCH[dtype]), dev(router), top, 1.0, ids, w, groups=groups[0] if groups else 0, keep=groups[1] if groups else 0,
                  renormalise=True, sigmoid=True, two_best=True)
    same = (ids.cpu().long() == chosen).all(dim=1)
    # (scores so near to one another that the last bits decide may stand the other way round)
    for t in torch.nonzero(~same).flatten().tolist():
        gap = (s[t, ids[t].cpu().long()] - s[t, chosen[t]]).abs().max()
        assert float(gap) < 1e-5 or groups, t
    assert float(same.double().mean()) > 0.98
    assert torch.allclose(w.cpu().to(F64)[same], weights[same], atol=1e-6)
    assert torch.allclose(w.cpu().sum(dim=1), torch.ones(n), atol=1e-5)


def test_groups_are_judged_by_their_two_largest():
    """A group with the one largest expert and nothing else loses against a group with two good ones."""
    from lia_rs_b200.kernels import ops
    z = torch.tensor([[3.0, -5.0, -5.0, 1.5, 1.4, -5.0], [-5.0, 3.0, 2.9, -5.0, 1.0, -5.0], [0.5, 0.5, 0.5, 0.5, 0.5, 0.5]])
    ids, w = torch.zeros(3, 2, dtype=torch.int32, device="cuda"), torch.zeros(3, 2, device="cuda")
    run = lambda **more: ops.moe_route(dev(torch.eye(3)), dev(z.T.contiguous()), 2, 1.0, ids, w, groups=2, keep=1, renormalise=True,
                                       sigmoid=True, **more)
    run(two_best=True)
    assert ids.cpu().tolist() == [[3, 4], [1, 2], [0, 1]]           # ties: the lower group, the lower expert
    pair = torch.sigmoid(torch.tensor([1.5, 1.4]))
    assert torch.allclose(w[0].cpu(), pair / pair.sum(), atol=1e-6)
    run(two_best=False)
    assert ids.cpu().tolist()[0][0] == 0                            # by the largest alone the first group would win


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hidden,ff,experts,top,groups,shared,n", [
    (72, 40, 6, 2, (3, 2), 24, 5), (64, 48, 10, 3, (5, 3), 96, 130), (128, 64, 8, 8, None, None, 33), (50, 30, 4, 1, (4, 1), 18, 17),
    (96, 32, 1, 1, None, 40, 9)])
def test_mixture_with_an_ungated_shared_expert(hidden, ff, experts, top, groups, shared, n, dtype):
    from lia_rs_b200.cache import CacheManager
    from lia_rs_b200.engine import StepEntry, StepRuntime
    from lia_rs_b200.parts import FEED_FORWARDS, KVCacheRequest, Runtime
    g = torch.Generator().manual_seed(hidden)
    mat = lambda rows, cols, s=1.0: bf(torch.randn(rows, cols, generator=g) * s / cols ** 0.5)
    w = {"router": mat(experts, hidden, 2.0)}
    for e in range(experts):
        w.update({f"e{e}.gate": mat(ff, hidden), f"e{e}.up": mat(ff, hidden), f"e{e}.down": mat(hidden, ff)})
    if shared:
        w.update({"shared.gate": mat(shared, hidden), "shared.up": mat(shared, hidden), "shared.down": mat(hidden, shared)})
    router = {"experts": experts, "top": top, **({"groups": {"count": groups[0], "keep": groups[1]}} if groups else {})}
    mlp = {"kind": "moe", "router": router, "expert": {"ff": ff}, **({"shared": {"ff": shared}} if shared else {})}
    params = {"hidden": hidden, "experts": experts, "top": top, "router_scale": 1.0, "intermediate": ff, "scores": "sigmoid",
              "groups": router.get("groups"), "group_score": "two_best", "renormalise": True,
              "shared": {"intermediate": shared} if shared else None, "shared_gated": False}
    h = bf(torch.randn(n, hidden, generator=g)).to(F64)
    fragile = torch.zeros(n, dtype=torch.bool)
    want = pb.expert_mixture(h, w, mlp, fragile)
    rt = Runtime(DEV, TORCH[dtype])
    cache = CacheManager({0: KVCacheRequest(1, 16)}, {}, 256, 2, 16, 256, TORCH[dtype], DEV)
    runtime = StepRuntime(cache, 1000, 256, DEV)
    part = FEED_FORWARDS["expert_mixture"](params, {"L." + k: v.to(DEV) for k, v in w.items()}, "L.", rt)
    slot = cache.admit()
    assert cache.ensure(slot, 0, n)
    ctx = runtime.begin([StepEntry(slot, [1] * n, 0, [])])
    for store in (True, False):
        residual = torch.ones(n, hidden, device=DEV)
        part.forward(ctx, dev(h, TORCH[dtype]), residual, 1.0, store=store)
        torch.cuda.synchronize()
        got = residual.cpu().to(F64) - (0.0 if store else 1.0)
        error = (got - want).abs()
        if dtype == "bfloat16":
            error = error[~fragile]
        assert float(error.max()) <= (2e-5 if dtype == "float32" else 4e-2) * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("hidden,n", [(50, 3), (256, 40)])
def test_the_stream_s_step(hidden, n):
    from lia_rs_b200.kernels import ops
    g = torch.Generator().manual_seed(n)
    x, x0, b = torch.randn(n, hidden, generator=g), torch.randn(n, hidden, generator=g), bf(torch.randn(hidden, generator=g))
    for first in (None, x0):
        for bias in (b, b.float(), None):
            got = dev(x.clone())
            ops.stream_sum(got, None if first is None else dev(first), None if bias is None else dev(bias))
            want = x + (0 if first is None else first)
            want = want + (0 if bias is None else bias.float())
            assert torch.allclose(got.cpu(), want, atol=1e-6)
