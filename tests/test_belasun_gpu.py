"""Belasun on the GPU engine against the plain CPU statement: mechanisms one by one, then whole models in 32-bit and bf16
through prompts, portions, decoding, mixed passes, reused slots and pages, snapshots, the serving scheduler and trace replay."""
import ctypes as C
import json
import os
import subprocess

import pytest
import torch

from belasun_oracle import (BANDS, MODELS, BelasunOracle, chunk_visible, expert, gelu_tanh, make_weights, masked_attention, mixture,
                            position_error, rms_norm, rotate_halves, rounding_spread, route, short_conv)
from test_stack_gpu import _ok, _stack, close, dev, feed, gen, limit

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16


# ---------------------------------------------------------------------------------------------------- models
_weights, _refs = {}, {}


def weights(name, dtype):
    """bf16 passes get weights whose routes do not hang on rounding."""
    if (name, dtype) not in _weights:
        _weights[name, dtype] = make_weights(MODELS[name], 1, steady=dtype == "bf16")
    return _weights[name, dtype]


def engine(name, dtype, **kw):
    from ds41rt_b200.models import belasun
    from ds41rt_b200.models.stack import StackEngine
    cfg, w = belasun.parse(MODELS[name], name), weights(name, dtype)
    return StackEngine(cfg, belasun.build_weights(cfg, lambda n: w[n], dev(), dtype),
                       **{"max_rows": 256, "slots": 4, "max_ctx": 1024, **kw})


def tokens(name, n, seed=0):
    return torch.randint(0, MODELS[name]["vocab"], (n,), generator=gen(seed)).tolist()


def reference(name, toks, dtype):
    """-> (logits, their rounding spread, layers, layer spreads)."""
    key = (name, tuple(toks), dtype)
    if key not in _refs:
        o = BelasunOracle(MODELS[name], weights(name, dtype))
        _refs[key] = o.forward(toks) + (rounding_spread(o, toks, 3) if dtype == "bf16" else (torch.full((len(toks),), 0.5),
                                        [torch.full((len(toks),), 0.5)] * len(MODELS[name]["layers"])))
    want, after, spread, layers = _refs[key]
    return want, spread, after, layers


PORTIONS = {"whole": [1024], "two": [2], "mixed": [70, 2, 3, 61, 64, 5, 65, 2, 130], "decode": [90, 1]}


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_prompts_portions_and_decoding_match_the_oracle(name, dtype):
    e = engine(name, dtype)
    toks = tokens(name, 230)
    want, spread, after, layer_spread = reference(name, toks, dtype)
    seen = []
    e.on_layer = lambda l, x: seen.append(x.cpu().double())
    e.cache.ensure(0, 230)
    e.set_rows(toks[:200], list(range(200)), [0] * 200)
    e.forward_rows(200, head=False)
    e.on_layer = None
    for got, ref, sp in zip(seen, after, layer_spread):
        close(got, ref[:200], dtype, sp[:200])
    e.cache.release(0)
    for sizes in PORTIONS.values():
        close(feed(e, 0, toks, 0, sizes), want, dtype, spread)
        e.cache.release(0)


@pytest.mark.parametrize("page", [16, 32, 128])
def test_other_page_sizes(page):
    e = engine("odd", "bf16", page_tokens=page)
    toks = tokens("odd", 230)
    want, spread = reference("odd", toks, "bf16")[:2]
    for sizes in ([1024], [90, 1], [100, 75, 2]):
        close(feed(e, 0, toks, 0, sizes), want, "bf16", spread)
        e.cache.release(0)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_first_tokens_of_a_sequence(dtype):
    e = engine("odd", dtype)
    for n in (1, 2, 3, 4, 5):
        toks = tokens("odd", n, seed=n)
        want, spread = reference("odd", toks, dtype)[:2]
        close(feed(e, 0, toks, 0, [1]), want, dtype, spread)
        e.cache.release(0)
        close(feed(e, 1, toks, 0, [8]), want, dtype, spread)
        e.cache.release(1)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_long_decoding(dtype):
    e = engine("odd", dtype)
    toks = tokens("odd", 330, seed=5)
    want, spread = reference("odd", toks, dtype)[:2]
    close(feed(e, 2, toks, 0, [80, 1]), want, dtype, spread)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_mixed_passes_of_unequal_requests(name, dtype):
    """Portions of four requests share passes; a request's logits are those it has alone."""
    e = engine(name, dtype, max_rows=128)
    reqs = {s: tokens(name, n, seed=20 + s) for s, n in enumerate((140, 33, 2, 75))}
    want = {s: reference(name, t, dtype)[:2] for s, t in reqs.items()}
    at = {s: 0 for s in reqs}
    got = {s: [] for s in reqs}
    plan = [{0: 40, 3: 30}, {0: 1, 1: 20, 3: 1}, {2: 1, 0: 60, 1: 12}, {3: 40, 2: 1, 1: 1}, {0: 39, 3: 4}]
    for step in plan:
        rows = []
        for s, n in step.items():
            assert e.cache.ensure(s, at[s] + n)
            rows += [(reqs[s][at[s] + i], at[s] + i, s) for i in range(n)]
            at[s] += n
        e.set_rows(*[list(x) for x in zip(*rows)])
        e.forward_rows(len(rows), head=False)
        lg, k = e.logits_at(list(range(len(rows)))).cpu().double(), 0
        for s, n in step.items():
            got[s].append(lg[k:k + n])
            k += n
    e.check_status()
    for s in reqs:
        assert at[s] == len(reqs[s])
        close(torch.cat(got[s]), want[s][0], dtype, want[s][1])


def test_slots_and_pages_are_used_again():
    """A small pool: requests come and go, later ones get pages in another order and slots with old states."""
    e = engine("odd", "f32", slots=2, n_pages=8, max_ctx=512)
    for i, (a, b) in enumerate([(200, 150), (90, 300), (310, 64), (65, 63)]):
        ta, tb = tokens("odd", a, seed=40 + i), tokens("odd", b, seed=50 + i)
        la, lb = feed(e, 0, ta[:60], 0, [60]), feed(e, 1, tb[:40], 0, [40])          # pages interleave
        la = torch.cat([la, feed(e, 0, ta[60:], 60, [50, 33])])
        lb = torch.cat([lb, feed(e, 1, tb[40:], 40, [90, 7])])
        for got, t in ((la, ta), (lb, tb)):
            want, spread = reference("odd", t, "f32")[:2]
            close(got, want, "f32", spread)
        for s in ((0, 1) if i % 2 else (1, 0)):
            e.cache.release(s)
    assert e.cache.free_pages == 8


def test_snapshots_continue_like_the_request_they_came_from():
    e = engine("odd", "f32")
    toks = tokens("odd", 260, seed=9)
    want, spread = reference("odd", toks, "f32")[:2]
    for n in (64, 100, 1):
        feed(e, 0, toks[:n], 0, [n])
        snap = e.cache.snapshot(0, n)
        feed(e, 0, tokens("odd", 50, seed=3), n, [50])              # the request goes on differently
        assert e.cache.restore(3, snap)
        close(feed(e, 3, toks[n:], n, [30, 1, 80]), want[n:], "f32", spread[n:])
        e.cache.drop_snapshot(snap)
        e.cache.release(0)
        e.cache.release(3)
    assert e.cache.free_pages == e.cache.n_pages


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_captured_decode_steps(dtype):
    from ds41rt_b200.runtime.session import DecodeSession
    e = engine("tiles", dtype)
    ses = DecodeSession(e)
    toks = [tokens("tiles", 60, seed=70 + s) for s in range(3)]
    want = [reference("tiles", t, dtype)[:2] for t in toks]
    for s in range(3):
        feed(e, s, toks[s][:20 + s], 0, [64])
        assert e.cache.ensure(s, 60)
    for i in range(30):
        pos = [20 + s + i for s in range(3)]
        ses.step([toks[s][p] for s, p in enumerate(pos)], pos, [0, 1, 2])
        lg = e.logits_rows(3).cpu()
        for s, p in enumerate(pos):
            err = float((lg[s].double() - want[s][0][p]).pow(2).mean().sqrt() / want[s][0].std())
            assert err < limit(dtype, float(want[s][1][p]))


def test_a_batch_larger_than_a_planned_pass():
    """Forty requests decode together: their experts go through the sorted form, in a captured pass too."""
    from ds41rt_b200.runtime.session import DecodeSession
    e = engine("odd", "bf16", slots=40, max_rows=64)
    toks = tokens("odd", 12, seed=8)
    want, spread = reference("odd", toks, "bf16")[:2]
    ses = DecodeSession(e)
    for s in range(40):
        assert e.cache.ensure(s, 12)
    for p, t in enumerate(toks):
        ses.step([t] * 40, [p] * 40, list(range(40)))
        lg = e.logits_rows(40).cpu().double()
        err = (lg - want[p]).pow(2).mean(-1).sqrt() / want.std()
        assert float(err.max()) < limit("bf16", float(spread[p]))
    e.check_status()


def _greedy(name, prompt, n):
    toks, o = list(prompt), BelasunOracle(MODELS[name], weights(name, "f32"))
    for _ in range(n):
        toks.append(int(o.forward(toks)[0][-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_session_and_scheduler():
    """The serving scheduler (admission, prompt passes, batched decode graphs, snapshot banks) generates what the oracle
    does, alone and with other requests, and a prompt that extends an earlier one continues from its snapshot."""
    from ds41rt_b200.runtime.session import DecodeSession
    from ds41rt_b200.serving.engine import GenRequest, NativeBackend
    from ds41rt_b200.serving.protocol import Sampling
    e = engine("odd", "f32", max_rows=64, slots=4)
    prompts = [tokens("odd", n, seed=90 + n) for n in (70, 5, 131)]
    want = [_greedy("odd", p, 10) for p in prompts]
    assert DecodeSession(e).generate(prompts[0], 10, slot=0) == want[0]
    e.cache.release(0)
    be = NativeBackend(e, eos=-1, concurrency=3, prefill_chunk=64)
    try:
        def submit(p):
            r = GenRequest(prompt_ids=p, max_tokens=10, sampling=Sampling(temperature=0.0))
            be.submit(r)
            return r

        def collect(r):
            toks, hit = [], 0
            while True:
                ev = r.events.get(timeout=60)
                assert ev.kind != "error", ev.message
                toks += ev.tokens
                hit = ev.usage.get("prompt_cache_hit_tokens", hit) if ev.kind == "ready" else hit
                if ev.kind == "finish":
                    return toks, hit

        assert [collect(r)[0] for r in [submit(p) for p in prompts]] == want
        longer = prompts[0] + want[0][:9] + tokens("odd", 9, seed=4)
        got, hit = collect(submit(longer))
        assert hit >= len(prompts[0]) and got == _greedy("odd", longer, 10)
        assert be.error is None
    finally:
        be.close()


def test_trace_replay_reads_a_checkpoint(tmp_path):
    from ds41rt_b200.loader.safetensors_io import write_safetensors
    doc = MODELS["odd"]
    a, b = tokens("odd", 90, seed=1), tokens("odd", 30, seed=2)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:70], "want": [0, 69]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[70:72], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[72:], "want": [17]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": b, "want": [29, 3]}], "end": ["y"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype, name in (("float32", "f32"), ("bfloat16", "bf16")):
        out = tmp_path / dtype
        out.mkdir()
        (out / "config.json").write_text(json.dumps(doc))
        write_safetensors(str(out / "model.safetensors"), {k: v.to(BF16) for k, v in weights("odd", name).items()})
        (wa, sa), (wb, sb) = reference("odd", a, name)[:2], reference("odd", b, name)[:2]
        r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(out), "--dtype", dtype, "--out",
                            str(out), "--max-tokens", "96"], input="".join(json.dumps(s) + "\n" for s in steps),
                           capture_output=True, text=True, timeout=240)
        assert r.returncode == 0, r.stderr[-800:]
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
        for n, (want, spread, rows) in {0: (wa, sa, [0, 69]), 2: (wa, sa, [89]), 3: (wb, sb, [29, 3])}.items():
            got = torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=F32).view(-1, doc["vocab"])
            for x, i in zip(got, rows):
                err = float((x.double() - want[i]).pow(2).mean().sqrt() / want.std())
                assert err < limit(name, float(spread[i]))


# ---------------------------------------------------------------------------------------------------- attention
class Pages:
    """One request's rows in scattered pages of a pool that is full of other values."""

    def __init__(self, n, page, row_len, dtype, seed=0):
        n_pages = -(-n // page)
        self.n, self.page, self.total = n, page, n_pages + 3
        self.order = torch.randperm(self.total, generator=gen(seed))[:n_pages]
        self.pool = torch.full((self.total * page, row_len), 7.0, dtype=dtype).cuda()
        self.table = torch.full((2, n_pages + 1), -1, dtype=torch.int32)
        self.table[1, :n_pages] = self.order.int()
        self.table = self.table.cuda()

    def at(self):
        """Pool row of every position."""
        pos = torch.arange(self.n)
        return (self.order[pos // self.page] * self.page + pos % self.page).cuda()


class Attention:
    """Random queries of the last `rows` positions over `n` keys; `far` = (row, key): the row's queries answer that key alone."""

    def __init__(self, H, G, D, V, n, rows, chunk, dtype, far=None, page=64, seed=0):
        g, r = gen(seed), lambda *s: torch.randn(*s, generator=gen(seed + len(s) + s[-1])).to(dtype).double()
        self.H, self.G, self.D, self.V, self.n, self.rows, self.chunk, self.dtype = H, G, D, V, n, rows, chunk, dtype
        self.q, self.k, self.v = r(rows, H, D), r(n, G, D), torch.randn(n, G, V, generator=g).to(dtype).double()
        self.gate = torch.randn(rows, H, generator=g)
        if far is not None:
            row, key = far
            u = torch.sign(self.k[key])
            self.k[key] = 2 * u
            self.q[row] = 2 * u.repeat_interleave(H // G, 0)
        self.dp, self.vp = (D + 15) // 16 * 16, (V + 15) // 16 * 16
        self.pages = Pages(n, page, G * (self.dp + self.vp), dtype, seed)
        pad = lambda x, w: torch.nn.functional.pad(x, (0, w - x.shape[-1])).flatten(1).to(dtype).cuda()
        self.pages.pool[self.pages.at()] = torch.cat([pad(self.k, self.dp), pad(self.v, self.vp)], 1)
        self.qd = pad(self.q, self.dp)
        self.scale = D ** -0.5

    def want(self):
        q = torch.zeros(self.n, self.H, self.D, dtype=torch.float64)
        q[self.n - self.rows:] = self.q
        o = masked_attention(q, self.k, self.v, self.scale, chunk_visible(self.n, self.chunk))[self.n - self.rows:]
        return o * torch.sigmoid(self.gate.double())[..., None]

    def run(self, kernel, splits=1):
        lib, S, k = _stack()
        rows = self.rows
        pos = torch.arange(self.n - rows, self.n, dtype=torch.int32).cuda()
        slot, G = torch.ones(rows, dtype=torch.int32).cuda(), self.gate.cuda()
        out = torch.full((rows, self.H * self.vp), 5.0, dtype=self.dtype).cuda()
        status = lib.new_status(dev())
        a = S.GroupAttendArgs()
        a.q, a.pool, a.page_table, a.row_pos, a.row_slot, a.out, a.status = (
            lib.ptr(t) for t in (self.qd, self.pages.pool, self.pages.table, pos, slot, out, status))
        a.gate, a.u, a.ld_q, a.scale = S.Proj(G, self.H).args(), S.NO_PROJ, self.H * self.dp, self.scale
        a.rows, a.heads, a.kv_heads, a.dim_pad, a.vdim_pad, a.chunk = rows, self.H, self.G, self.dp, self.vp, self.chunk or 0
        a.taps, a.slots, a.n_splits, a.ld_out, a.max_pages = 1, 2, splits, self.H * self.vp, self.pages.table.shape[1]
        a.page_tokens, a.f32, a.n_pages, a.pos0 = self.pages.page, int(self.dtype == F32), self.pages.total, self.n - rows
        _ok(getattr(k, f"ds41_group_{kernel}")(C.byref(a), lib.stream()))
        lib.raise_on_status(status)
        got = out.cpu().double().view(rows, self.H, self.vp)
        assert not got[..., self.V:].any()
        return got[..., :self.V]


def test_attention_of_more_blocks_than_multiprocessors():
    for shape in ((6, 2, 20, 24), (8, 1, 128, 128), (4, 2, 48, 80)):
        c = Attention(*shape, 260, 200, 100, BF16, seed=7)
        for splits in (1, 2):
            torch.testing.assert_close(c.run("attend", splits), c.want(), rtol=0.03, atol=0.03)


SHAPES = [(6, 2, 20, 24), (3, 3, 64, 64), (8, 1, 128, 128), (40, 2, 48, 80), (1, 1, 16, 200)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("splits", [1, 3, 16])
@pytest.mark.parametrize("shape", SHAPES)
def test_attention_over_pages_and_chunks(shape, splits, dtype):
    """Rows around chunk borders: the last position of a chunk, the first of the next, the middle; or everything visible."""
    tol = 2e-5 if dtype == F32 else 0.03
    for n, rows, chunk in ((130, 5, 128), (257, 3, 64), (300, 2, None), (90, 4, 1), (75, 3, 1000)):
        c = Attention(*shape, n, rows, chunk, dtype, seed=n)
        torch.testing.assert_close(c.run("attend", splits), c.want(), rtol=tol, atol=tol)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("kernel,rows", [("attend", 3), ("prefill", 200)])
def test_one_key_stands_out_at_the_edge_of_a_chunk(kernel, rows, dtype):
    """A key that answers a row's queries far above all others: the chunk's first position counts, the one before does not."""
    if kernel == "prefill" and dtype == F32:
        pytest.skip("the long-pass form is bf16")
    n, chunk = 300, 150
    for row, key, seen in ((rows - 1, 150, True), (rows - 1, 149, False), (rows - 1, 299, True), (rows - 2, 299, False),
                           (rows - 1, 192, True), (rows - 1, 255, True)):
        c = Attention(4, 2, 64, 32, n, rows, chunk, dtype, far=(row, key), seed=key)
        got, want = c.run(kernel), c.want()
        torch.testing.assert_close(got, want, rtol=0.03, atol=0.03)
        only = c.v[key].repeat_interleave(2, 0) * torch.sigmoid(c.gate[row].double())[:, None]
        cos = torch.nn.functional.cosine_similarity(got[row], only, dim=-1)
        assert (cos > 0.98).all() if seen else (cos < 0.9).any()


@pytest.mark.parametrize("shape", [(6, 2, 20, 24), (5, 1, 64, 128), (3, 3, 128, 112), (2, 1, 192, 64), (4, 4, 16, 16)])
@pytest.mark.parametrize("page", [32, 64, 128])
def test_prompt_attention_over_pages_and_chunks(shape, page):
    """Long passes: pairs of heads, an odd head, pairs of row tiles; chunks shorter and longer than a tile, off its grid."""
    for n, rows, chunk in ((129, 129, None), (300, 257, 64), (520, 300, 100), (700, 65, 512), (384, 384, 37), (200, 200, 1)):
        c = Attention(*shape, n, rows, chunk, BF16, page=page, seed=n)
        torch.testing.assert_close(c.run("prefill"), c.want(), rtol=0.03, atol=0.03)


class Post:
    """Projections of one request fed in portions through attn_post, followed by the attention launch that keeps the
    convolution's inputs, -> (queries, keys, values) of all positions."""

    def __init__(self, T, H, G, D, V, taps, rot, dtype=F32, seed=0, norm=True, packed=False):
        """packed: the projection is one bf16 matrix (long passes), else two split-K planes."""
        g = gen(seed)
        self.T, self.H, self.G, self.D, self.V, self.taps, self.rot, self.dtype = T, H, G, D, V, taps, rot, dtype
        self.w = [torch.randn(h * d, max(taps, 1), generator=g) for h, d in ((H, D), (G, D), (G, V))]
        self.u = [torch.randn(T, h * d, generator=g) for h, d in ((H, D), (G, D), (G, V))]
        self.packed = packed
        if packed:
            self.u = [x.to(BF16).float() for x in self.u]
        self.nq, self.nk = torch.rand(H * D, generator=g) + 0.5, torch.rand(G * D, generator=g) + 0.5
        self.norm = norm

    def want(self, eps):
        q, k, v = (short_conv(u.double(), w.double()) if self.taps else u.double() for u, w in zip(self.u, self.w))
        if self.norm:
            q, k = rms_norm(q, self.nq.double(), eps), rms_norm(k, self.nk.double(), eps)
        pos, T = torch.arange(self.T), self.T
        turn = lambda x: rotate_halves(x, pos, self.rot) if self.rot else x
        return turn(q.view(T, self.H, self.D)), turn(k.view(T, self.G, self.D)), v.view(T, self.G, self.V)

    def run(self, sizes, eps, splits=2, page=16):
        from ds41rt_b200.config import rope_inv_freq
        from ds41rt_b200.models import belasun
        lib, S, k = _stack()
        dp, vp = S.ceil_to(self.D, 16), S.ceil_to(self.V, 16)
        H, G, T = self.H, self.G, self.T
        pads = lambda x, n, d, p: S.pad_heads(x.t().contiguous(), n, d, p).t()
        heads = ((H, self.D, dp), (G, self.D, dp), (G, self.V, vp))
        u = torch.cat([pads(x, *h) for x, h in zip(self.u, heads)], 1)
        cols = u.shape[1]
        planes = (u.to(BF16)[None] if self.packed else torch.stack([u * 0.25, u * 0.75])).contiguous().cuda()
        conv = torch.cat([S.pad_heads(w, *h) for w, h in zip(self.w, heads)], 0).t().contiguous().cuda()
        nq, nk = (S.pad_heads(x, *h).cuda() for x, h in zip((self.nq, self.nk), heads))
        rot_dim, rope = belasun._rope(self.rot, "rot") if self.rot else (0, None)
        freq = torch.tensor(rope_inv_freq(rope, rot_dim) if rope else [0.0], dtype=F32).cuda()
        back = max(self.taps, 1) - 1
        state = torch.full((2, max(back, 1), cols), float("nan")).cuda()                      # what an old request left
        pages = Pages(T, page, G * (dp + vp), self.dtype)
        out_q, at, i = [], 0, 0
        while at < T:
            n = min(sizes[min(i, len(sizes) - 1)], T - at)
            x = planes[:, at:at + n].contiguous()
            pos = torch.arange(at, at + n, dtype=torch.int32).cuda()
            slot = torch.ones(n, dtype=torch.int32).cuda()
            q, o = torch.zeros(n, H * dp, dtype=self.dtype).cuda(), torch.zeros(n, H * vp, dtype=self.dtype).cuda()
            a = S.AttnPostArgs()
            a.u = (S.Proj(x, cols) if self.packed else S.Proj(x, cols, 2, n * cols)).args()
            a.conv, a.q_norm, a.k_norm, a.freq, a.state, a.q, a.pool = (lib.ptr(t) for t in (
                conv if self.taps else None, nq if self.norm else None, nk if self.norm else None, freq, state, q, pages.pool))
            a.page_table, a.row_pos, a.row_slot, a.ld_q, a.eps = lib.ptr(pages.table), lib.ptr(pos), lib.ptr(slot), H * dp, eps
            a.rows, a.heads, a.kv_heads, a.dim, a.dim_pad, a.vdim_pad, a.rot_dim = n, H, G, self.D, dp, vp, rot_dim
            a.taps, a.slots, a.max_pages, a.page_tokens, a.f32 = back + 1, 2, pages.table.shape[1], page, int(self.dtype == F32)
            _ok(k.ds41_attn_post(C.byref(a), lib.stream()))
            b = S.GroupAttendArgs()
            b.q, b.pool, b.page_table, b.row_pos, b.row_slot, b.out, b.state = (
                lib.ptr(t) for t in (q, pages.pool, pages.table, pos, slot, o, state))
            b.gate, b.u, b.ld_q, b.scale = S.NO_PROJ, a.u, H * dp, 1.0
            b.rows, b.heads, b.kv_heads, b.dim_pad, b.vdim_pad, b.chunk, b.taps, b.slots = n, H, G, dp, vp, 0, back + 1, 2
            b.n_splits, b.ld_out, b.max_pages, b.page_tokens, b.f32 = splits, H * vp, a.max_pages, page, a.f32
            b.n_pages = pages.total
            _ok(k.ds41_group_attend(C.byref(b), lib.stream()))
            torch.cuda.synchronize()
            out_q.append(q.cpu().double())
            at, i = at + n, i + 1
        assert torch.isnan(state[0]).all() and (back == 0 or T < back or torch.isfinite(state[1]).all())
        q = torch.cat(out_q).view(T, H, dp)
        rows = pages.pool[pages.at()].cpu().double()
        kk, v = rows[:, :G * dp].view(T, G, dp), rows[:, G * dp:].view(T, G, vp)
        assert not q[..., self.D:].any() and not kk[..., self.D:].any() and not v[..., self.V:].any()
        return q[..., :self.D], kk[..., :self.D], v[..., :self.V]


@pytest.mark.parametrize("form", [(F32, False), (BF16, False), (BF16, True)])
@pytest.mark.parametrize("sizes", [[100], [1], [2], [7, 1, 3, 2, 1, 1, 20], [40, 2, 38]])
@pytest.mark.parametrize("shape", [dict(H=6, G=2, D=20, V=24, taps=4, rot=dict(base=40.0, dims=12, scaling=BANDS)),
                                   dict(H=1, G=1, D=16, V=16, taps=1, rot=dict(base=9.0, dims=16)),
                                   dict(H=20, G=4, D=128, V=64, taps=2, rot=dict(base=100.0, dims=128)),
                                   dict(H=40, G=5, D=128, V=128, taps=3, rot=dict(base=100.0, dims=64)),
                                   dict(H=3, G=3, D=10, V=40, taps=7, rot=None, norm=False),
                                   dict(H=2, G=1, D=34, V=16, taps=0, rot=dict(base=100.0, dims=2))])
def test_convolution_norm_rotation_and_cache_rows(shape, sizes, form):
    """Every form of the launch: 32-bit or bf16 results, few rows or a block of them, portions shorter than the taps."""
    dtype, packed = form
    c = Post(80, **shape, dtype=dtype, seed=shape["H"], packed=packed)
    tol = 3e-5 if dtype == F32 else 1e-2
    for got, want in zip(c.run(sizes, 1e-3), c.want(1e-3)):
        torch.testing.assert_close(got, want, rtol=tol, atol=tol)


# ---------------------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("rows,experts,top", [(1, 1, 1), (3, 5, 2), (9, 40, 6), (32, 512, 8), (300, 100, 32), (5, 33, 33 - 1)])
def test_router_choices_weights_and_plan(rows, experts, top):
    lib, S, k = _stack()
    g = gen(experts)
    z, b = torch.randn(2, rows, experts, generator=g), torch.randn(experts, generator=g)
    z[:, 0] = z[:, 0].round()                                  # ties: the lower index wins
    b[: experts // 2] = 0.0
    if rows > 2:
        z[0, 2, 0] += 400.0                                    # one logit far above: the other weights vanish
    slot = torch.arange(rows, dtype=torch.int32)
    slot[rows // 2:rows // 2 + (rows > 1)] = -1
    most = min(experts, rows * top)
    Z, B, SL = z.cuda(), b.cuda(), slot.cuda()
    i32, f32 = (lambda *s: torch.full(s, -7, dtype=torch.int32).cuda()), (lambda *s: torch.full(s, -7.0).cuda())
    ids, wt, active, n_act, row_w, slot_of = i32(rows, top), f32(rows, top), i32(most), i32(1), f32(most, rows + 3), i32(rows, top)
    ticket = torch.zeros(1, dtype=torch.int32).cuda()
    a = S.RouteArgs()
    a.z = S.Proj(Z, experts, 2, rows * experts).args()
    a.bias, a.row_slot, a.ids, a.weights = (lib.ptr(t) for t in (B, SL, ids, wt))
    a.active, a.n_active, a.row_w, a.slot_of, a.ticket = (lib.ptr(t) for t in (active, n_act, row_w, slot_of, ticket))
    a.rows, a.experts, a.top, a.max_active, a.row_w_ld = rows, experts, top, most, rows + 3
    for _ in range(2):                                         # the ticket is left ready for the next launch
        _ok(k.ds41_route_softmax(C.byref(a), lib.stream()))
        logits = (z[0] + z[1]) + b
        best = torch.sort(logits, dim=-1, descending=True, stable=True)
        want_ids, want_w = best.indices[:, :top].clone(), torch.softmax(best.values[:, :top].double(), -1)
        want_ids[slot < 0] = -1
        assert torch.equal(ids.cpu().long(), want_ids)
        torch.testing.assert_close(wt.cpu().double(), want_w, rtol=1e-5, atol=1e-9)
        live = (wt.cpu() > 0) & (slot >= 0)[:, None]
        used = sorted(set(want_ids[live].tolist()))
        assert int(n_act) == len(used) and active.cpu()[:len(used)].tolist() == used and int(ticket) == 0
        dense = torch.zeros(most, rows + 3)
        for r_, k_ in live.nonzero().tolist():
            dense[used.index(int(want_ids[r_, k_])), r_] = wt.cpu()[r_, k_]
        assert torch.equal(row_w.cpu(), dense)
        assert torch.equal(slot_of.cpu() >= 0, live)
        assert all(used[s] == i for s, i in zip(slot_of.cpu()[live].tolist(), want_ids[live].tolist()))


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("rows", [1, 3, 32, 33, 150])
def test_experts_planned_and_sorted(rows, dtype):
    """One mixture on given input rows, some of which belong to nobody, summed and added by the residual step."""
    e = engine("odd", dtype)
    W, ml = 90, MODELS["odd"]["layers"][0]["mlp"]
    lw, w = e.w.layers[0], weights("odd", dtype)
    h = torch.randn(rows, W, generator=gen(rows)).to(BF16).float()
    h[:, :7] *= 4                                              # clear routes (the code columns of the steady weights)
    idle = rows // 2 if rows > 2 else -1
    e.set_rows(None, [0] * rows, [-1 if i == idle else i for i in range(rows)])
    e.h.zero_()
    e.h[:rows, :W] = h.cuda().to(e.h.dtype)
    y, gate = lw.mlp.run(e, rows)
    x = torch.randn(rows, e.ldx, generator=gen(1)).cuda()
    out = torch.zeros_like(x)
    e._resid(rows, y=y, gate=gate, x_in=x, x_out=out)
    e.check_status()
    got = (out - x).cpu().double()[:, :W]
    want = mixture(h.double(), {k: v.double() for k, v in w.items()}, "l0.mlp.", ml)
    if idle >= 0:
        want[idle] = 0
    tol = 2e-5 if dtype == "f32" else 0.02
    scale = float(want.abs().max())
    torch.testing.assert_close(got / scale, want / scale, rtol=tol, atol=tol)
    raw = e.h[:rows, :W].float().cpu()                         # with no norm to come the next sublayer reads the stream itself
    torch.testing.assert_close(raw, out.cpu()[:, :W], rtol=1e-2 if dtype == "bf16" else 0, atol=1e-2 if dtype == "bf16" else 0)


def test_the_expert_activation_is_cut_where_it_should_be():
    """Gate and up values around and far beyond the limits, 32-bit activation."""
    lib, S, k = _stack()
    v = torch.tensor([-50.0, -2.1, -1.9, -0.3, 0.0, 0.4, 1.9, 2.1, 50.0])
    g, u = torch.meshgrid(v, v, indexing="ij")
    x = torch.cat([g.reshape(1, -1), u.reshape(1, -1)], 1).cuda()
    n = g.numel()
    act, w, one = torch.zeros(1, n).cuda(), torch.full((1, 1), 0.5).cuda(), torch.ones(1, dtype=torch.int32).cuda()
    _ok(k.ds41_gated_act(lib.ptr(x), 2 * n, n, lib.ptr(w), 1, lib.ptr(one), 1, 1, n, C.c_float(2.0), C.c_float(1.702),
                         C.c_float(1.0), lib.ptr(act), n, lib.stream()))
    eye = {"gate": torch.ones(1, 1, dtype=torch.float64), "down": torch.ones(1, 1, dtype=torch.float64)}
    want = [float(expert(torch.ones(1, 1, dtype=torch.float64), dict(eye, gate=eye["gate"] * a, up=eye["gate"] * b), "", 2.0))
            for a, b in zip(g.reshape(-1).double(), u.reshape(-1).double())]
    torch.testing.assert_close(act.cpu().double()[0], 0.5 * torch.tensor(want, dtype=torch.float64), rtol=1e-5, atol=1e-6)


# ---------------------------------------------------------------------------------------------------- token input, logits
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n,col", [(1, 3), (10, 20), (300, 0)])
def test_token_input_reads_the_layers_own_part(n, col, dtype):
    lib, S, k = _stack()
    g = gen(n)
    z, table = torch.randn(2, 5, n, generator=g), torch.randn(11, col + n + 4, generator=g).to(BF16)
    toks = torch.tensor([0, 10, 4, 11, -1], dtype=torch.int32)             # two that the table does not have
    ld = S.ceil_to(n, 8)
    out = torch.full((5, ld), 9.0, dtype=dtype).cuda()
    Z, E, T = z.cuda(), table.cuda(), toks.cuda()
    _ok(k.ds41_side_act(C.byref(S.Proj(Z, n, 2, 5 * n).args()), lib.ptr(T), lib.ptr(E), C.c_longlong(table.shape[1]), col, 11, 5, n,
                        lib.ptr(out), ld, int(dtype == F32), lib.stream()))
    want = torch.zeros(5, ld, dtype=torch.float64)
    want[:3, :n] = gelu_tanh(z.double().sum(0))[:3] * table.double()[toks[:3].long(), col:col + n]
    tol = 1e-5 if dtype == F32 else 1e-2
    torch.testing.assert_close(out.cpu().double(), want, rtol=tol, atol=tol)


@pytest.mark.parametrize("rows,W", [(3, 90), (2, 2048), (40, 2048)])
def test_result_norm_is_an_rms_norm_whatever_the_models_norm_is(rows, W):
    lib, S, k = _stack()
    g = gen(W)
    y, x, pw = torch.randn(rows, W, generator=g) + 0.7, torch.randn(rows, W, generator=g), torch.randn(W, generator=g)
    Lw = S.ceil_to(W, 8)
    pad = lambda t: torch.nn.functional.pad(t, (0, Lw - W)).cuda()
    Y, X, PW, out = pad(y), pad(x), pw.cuda(), torch.zeros(rows, Lw).cuda()
    a = S.ResidArgs()
    a.y, a.gate, a.post_w, a.x_in, a.x_out = S.Proj(Y, Lw).args(), S.NO_PROJ, lib.ptr(PW), lib.ptr(X), lib.ptr(out)
    a.ldx, a.ldh, a.rows, a.W, a.norm_kind, a.post_rms, a.eps, a.f32 = Lw, Lw, rows, W, 0, 1, 1e-5, 1
    _ok(k.ds41_resid_step(C.byref(a), lib.stream()))
    want = x.double() + rms_norm(y.double(), pw.double(), 1e-5)
    torch.testing.assert_close(out[:, :W].cpu().double(), want, rtol=2e-5, atol=2e-5)


def test_soft_cap_in_both_forms():
    lib, S, k = _stack()
    from ds41rt_b200.ops import gemm as G
    g = gen(5)
    w, x = (torch.randn(300, 64, generator=g) * 2).to(BF16), torch.randn(7, 64, generator=g).to(BF16)
    raw = x.double() @ w.double().T
    want = 6.0 * torch.tanh(raw / 6.0)
    assert float((raw - want).abs().max()) > 10
    out, Wd, X = torch.zeros(7, 300).cuda(), w.cuda(), x.cuda()
    G.gemm_raw(Wd, X, out, 300, 7, 64, lda=64, ldb=64, ldo=300, out_mode=3, softcap=6.0)
    torch.testing.assert_close(out.cpu().double(), want, rtol=1e-4, atol=1e-4)
    out2 = raw.float().cuda()
    _ok(k.ds41_softcap_rows(lib.ptr(out2), C.c_longlong(out2.numel()), C.c_float(6.0), lib.stream()))
    torch.testing.assert_close(out2.cpu().double(), want, rtol=1e-5, atol=1e-5)


def test_bad_arguments_are_refused_on_the_host():
    lib, S, k = _stack()
    for fn, args in (("attn_post", S.AttnPostArgs), ("group_attend", S.GroupAttendArgs), ("group_prefill", S.GroupAttendArgs),
                     ("route_softmax", S.RouteArgs)):
        assert getattr(k, f"ds41_{fn}")(C.byref(args()), lib.stream()) != 0 and getattr(k, f"ds41_{fn}")(None, lib.stream()) != 0
    c = Attention(4, 2, 64, 32, 100, 3, 64, BF16)
    with pytest.raises(AssertionError):
        c.run("attend", splits=17)
    c.pages.page = 48                                                      # a page size the long-pass form does not take
    with pytest.raises(AssertionError):
        c.run("prefill")
