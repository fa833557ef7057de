"""Genesun on the GPU engine against the plain CPU statement: mechanisms one by one, then whole models in 32-bit and bf16
through prompts, portions, decoding, mixed passes, reused slots and pages, snapshots, the serving scheduler and trace replay."""
import ctypes as C
import json
import math
import os
import subprocess
import sys

import pytest
import torch

from genesun_oracle import (MODELS, GenesunOracle, layer_norm, make_weights, mlstm_scan, polynorm, position_error, rms_unit,
                            rotate_pairs, rounding_spread, sink_softmax_attention)

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16


def dev():
    return torch.device("cuda", 0)


def gen(seed=0):
    return torch.Generator().manual_seed(seed)


# ---------------------------------------------------------------------------------------------------- models
_cache = {}


def oracle(name, seed=1):
    if (name, seed) not in _cache:
        doc = MODELS[name]
        _cache[name, seed] = (doc, make_weights(doc, seed))
    doc, w = _cache[name, seed]
    return GenesunOracle(doc, w)


def engine(name, dtype, seed=1, **kw):
    from ds41rt_b200.models import genesun
    from ds41rt_b200.models.stack import StackEngine
    oracle(name, seed)
    doc, w = _cache[name, seed]
    cfg = genesun.parse(doc, name)
    kw = {"max_rows": 256, "slots": 4, "max_ctx": 1024, **kw}
    return StackEngine(cfg, genesun.build_weights(cfg, lambda n: w[n], dev(), dtype), **kw)


def tokens(name, n, seed=0):
    return torch.randint(0, MODELS[name]["vocab"], (n,), generator=gen(seed)).tolist()


def feed(e, slot, toks, start, sizes):
    """Run `toks` from position `start` in portions of `sizes` (the last size repeats) -> logits of every position."""
    out, i, k = [], 0, 0
    assert e.cache.ensure(slot, start + len(toks))
    while i < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - i)
        e.set_rows(toks[i:i + n], list(range(start + i, start + i + n)), [slot] * n)
        e.forward_rows(n, head=False)
        out.append(e.logits_at(list(range(n))).cpu().double())
        i, k = i + n, k + 1
    e.check_status()
    return torch.cat(out)


def limit(dtype, spread):
    """Allowed difference at a position whose bf16 rounding spread is known: a floor plus a multiple of what rounding does
    there (a 32-bit pass rounds 2^16 times finer; the factor leaves room for sums over many terms)."""
    return 2e-5 + 4e-4 * spread if dtype == "f32" else 0.03 + 3 * spread


def close(got, want, dtype, spread):
    err, lim = position_error(got, want), limit(dtype, spread)
    bad = err / lim
    assert torch.isfinite(got).all() and float(bad.max()) < 1, \
        f"worst {float(err[bad.argmax()]):.3e} (limit {float(lim[bad.argmax()]):.3e}) at row {int(bad.argmax())}"


_refs = {}


def reference(name, toks):
    """-> (logits, their rounding spread, layers, layer spreads)."""
    key = (name, tuple(toks))
    if key not in _refs:
        o = oracle(name)
        _refs[key] = o.forward(toks) + rounding_spread(o, toks)
    want, after, spread, layers = _refs[key]
    return want, spread, after, layers


PORTIONS = {"whole": [1024], "two": [2], "mixed": [70, 2, 3, 61, 64, 5, 65, 2, 130], "decode": [90, 1]}


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_prompts_portions_and_decoding_match_the_oracle(name, dtype):
    e = engine(name, dtype)
    toks = tokens(name, 230)
    want, spread, after, layer_spread = reference(name, toks)
    e.on_layer = lambda l, x: seen.append(x.cpu().double())
    seen = []
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


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_first_tokens_of_a_sequence(dtype):
    e = engine("plain", dtype)
    for n in (1, 2, 3):
        toks = tokens("plain", n, seed=n)
        want, spread = reference("plain", toks)[:2]
        close(feed(e, 0, toks, 0, [1]), want, dtype, spread)
        e.cache.release(0)
        close(feed(e, 1, toks, 0, [8]), want, dtype, spread)
        e.cache.release(1)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_long_decoding(dtype):
    e = engine("odd", dtype)
    toks = tokens("odd", 400, seed=5)
    want, spread = reference("odd", toks)[:2]
    close(feed(e, 2, toks, 0, [100, 1]), want, dtype, spread)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_mixed_passes_of_unequal_requests(name, dtype):
    """Portions of four requests share passes; a request's logits are those it has alone."""
    e = engine(name, dtype, max_rows=128)
    reqs = {s: tokens(name, n, seed=20 + s) for s, n in enumerate((140, 33, 2, 75))}
    want = {s: reference(name, t)[:2] for s, t in reqs.items()}
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
            want, spread = reference("odd", t)[:2]
            close(got, want, "f32", spread)
        for s in ((0, 1) if i % 2 else (1, 0)):
            e.cache.release(s)
    assert e.cache.free_pages == 8


def test_snapshots_continue_like_the_request_they_came_from():
    e = engine("odd", "f32")
    toks = tokens("odd", 260, seed=9)
    want, spread = reference("odd", toks)[:2]
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
def test_captured_decode_steps_advance_the_state_once(dtype):
    from ds41rt_b200.runtime.session import DecodeSession
    e = engine("tiles", dtype)
    ses = DecodeSession(e)
    toks = [tokens("tiles", 60, seed=70 + s) for s in range(3)]
    want = [reference("tiles", t)[:2] for t in toks]
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


def _greedy(name, prompt, n):
    toks, o = list(prompt), oracle(name)
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
    want = [_greedy("odd", p, 12) for p in prompts]
    assert DecodeSession(e).generate(prompts[0], 12, slot=0) == want[0]
    e.cache.release(0)
    be = NativeBackend(e, eos=-1, concurrency=3, prefill_chunk=64)
    try:
        def submit(p, n=12):
            r = GenRequest(prompt_ids=p, max_tokens=n, sampling=Sampling(temperature=0.0))
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
        assert be.totals["graph_rounds"] > 0
        longer = prompts[0] + want[0][:11] + tokens("odd", 9, seed=4)
        got, hit = collect(submit(longer))
        assert hit >= len(prompts[0]) and got == _greedy("odd", longer, 12)
        shared = prompts[2][:100] + tokens("odd", 20, seed=6)             # only a leading part is shared: run from the start
        got, hit = collect(submit(shared))
        assert hit == 0 and got == _greedy("odd", shared, 12)
        assert be.error is None
    finally:
        be.close()


def test_trace_replay_reads_a_checkpoint(tmp_path):
    from ds41rt_b200.loader.safetensors_io import write_safetensors
    doc = MODELS["odd"]
    oracle("odd")
    w = _cache["odd", 1][1]
    (tmp_path / "config.json").write_text(json.dumps(doc))
    write_safetensors(str(tmp_path / "model.safetensors"), {k: v.to(BF16) for k, v in w.items()})
    a, b = tokens("odd", 90, seed=1), tokens("odd", 30, seed=2)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:70], "want": [0, 69]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[70:72], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[72:], "want": [17]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": b, "want": [29, 3]}], "end": ["y"]}]
    (wa, sa), (wb, sb) = reference("odd", a)[:2], reference("odd", b)[:2]
    expect = {0: (wa, sa, [0, 69]), 2: (wa, sa, [89]), 3: (wb, sb, [29, 3])}
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype, name in (("float32", "f32"), ("bfloat16", "bf16")):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out",
                            str(out), "--max-tokens", "96"], input="".join(json.dumps(s) + "\n" for s in steps),
                           capture_output=True, text=True, timeout=240)
        assert r.returncode == 0, r.stderr[-800:]
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
        assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
        for n, (want, spread, rows) in expect.items():
            got = torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=F32).view(-1, doc["vocab"])
            for x, i in zip(got, rows):
                err = float((x.double() - want[i]).pow(2).mean().sqrt() / want.std())
                assert err < limit(name, float(spread[i]))


# ---------------------------------------------------------------------------------------------------- mechanisms
def _stack():
    from ds41rt_b200.ops import lib
    from ds41rt_b200.ops import stack as S
    return lib, S, lib.kernels()


def _ok(err):
    assert err == 0, f"cudaError {err}"


@pytest.mark.parametrize("rows,W,kind", [(3, 52, 0), (4, 90, 0), (33, 1032, 0), (5, 1032, 1), (3, 1501, 0), (2, 4096, 0),
                                         (40, 4096, 0), (40, 9000, 1), (2, 20001, 0)])
def test_residual_step(rows, W, kind):
    lib, S, k = _stack()
    g = gen(W)
    r = lambda *s: torch.randn(*s, generator=g)
    y, gt, b, pw, nw, x = r(2, rows, W), r(2, rows, W), r(W), r(W), r(W), r(rows, W)
    kept, mix, eps = r(3, rows, W), r(4), 1e-5
    norm = layer_norm if kind == 0 else (lambda v, w, e: rms_unit(v, e) * w)
    d = lambda t: t.double()
    full = d(x) + norm(d(y).sum(0) * torch.sigmoid(d(gt).sum(0) + d(b)), d(pw), eps)
    avg = sum(m * t for m, t in zip(d(mix), [*d(kept), full]))
    L = S.ceil_to(W, 8)

    def wide(t):                    # rows padded with values that must not count
        o = torch.full(t.shape[:-1] + (L,), float("nan"), device="cuda")
        o[..., :W] = t.cuda()
        return o

    Y, GT, X, KEPT = map(wide, (y, gt, x, kept))
    B, PW, NW, MIX = (t.cuda() for t in (b, pw, nw, mix))
    out, x_avg, h = (torch.zeros(rows, L).cuda() for _ in range(3))
    a = S.ResidArgs()
    a.y, a.gate = S.Proj(Y, L, 2, rows * L).args(), S.Proj(GT, L, 2, rows * L).args()
    a.gate_bias, a.post_w, a.next_w, a.x_in, a.x_out = (lib.ptr(t) for t in (B, PW, NW, X, out))
    a.mix, a.kept, a.kept_stride, a.n_mix, a.x_avg = lib.ptr(MIX), lib.ptr(KEPT), rows * L, 4, lib.ptr(x_avg)
    a.h, a.ldh, a.ldx, a.rows, a.W, a.norm_kind, a.eps, a.f32 = lib.ptr(h), L, L, rows, W, kind, eps, 1
    _ok(k.ds41_resid_step(C.byref(a), lib.stream()))
    torch.testing.assert_close(out[:, :W].cpu().double(), full, rtol=2e-5, atol=2e-5)
    torch.testing.assert_close(x_avg[:, :W].cpu().double(), avg, rtol=2e-5, atol=2e-5)
    torch.testing.assert_close(h[:, :W].cpu().double(), norm(avg, d(nw), eps), rtol=2e-5, atol=5e-5)
    # start from the embedding, bf16 output
    E = r(17, W).to(BF16)
    toks = torch.randint(0, 17, (rows,), generator=g)
    a = S.ResidArgs()
    a.y = a.gate = S.NO_PROJ
    te, tt, hb = wide(E).to(BF16), toks.int().cuda(), torch.zeros(rows, L, dtype=BF16).cuda()
    a.tokens, a.embed, a.embed_ld, a.vocab, a.x_out, a.next_w = lib.ptr(tt), lib.ptr(te), L, 17, lib.ptr(out), lib.ptr(NW)
    a.h, a.ldh, a.ldx, a.rows, a.W, a.norm_kind, a.eps = lib.ptr(hb), L, L, rows, W, kind, eps
    _ok(k.ds41_resid_step(C.byref(a), lib.stream()))
    assert torch.equal(out[:, :W].cpu(), E[toks].float())
    torch.testing.assert_close(hb[:, :W].cpu().double(), norm(d(E[toks]), d(nw), eps), rtol=1e-2, atol=1e-2)


@pytest.mark.parametrize("ff", [37, 640, 5000])
def test_polynorm_and_gates(ff):
    lib, S, k = _stack()
    g = gen(ff)
    z, coef, ld = torch.randn(2, 4, ff, generator=g), torch.tensor([0.7, -0.4, 0.3, 0.2]), S.ceil_to(ff, 8)
    out = torch.zeros(4, ld).cuda()
    Z, Cf = torch.full((2, 4, ld), float("nan")).cuda(), coef.cuda()        # what lies beyond the row does not count
    Z[..., :ff] = z.cuda()
    _ok(k.ds41_polynorm(C.byref(S.Proj(Z, ld, 2, 4 * ld).args()), lib.ptr(Cf), 4, ff, C.c_float(1e-5), lib.ptr(out), ld, 1,
                        lib.stream()))
    torch.testing.assert_close(out[:, :ff].cpu().double(), polynorm(z.double().sum(0), coef.double(), 1e-5), rtol=3e-5,
                               atol=3e-5)
    n, out = ff // 4 * 4, torch.zeros(4, ld).cuda()
    _ok(k.ds41_gate_mul(C.byref(S.Proj(Z[0], ld).args()), C.byref(S.Proj(Z[1], ld).args()), 4, n, lib.ptr(out), ld, 1,
                        lib.stream()))
    torch.testing.assert_close(out[:, :n].cpu(), (z[0] * torch.sigmoid(z[1]))[:, :n], rtol=1e-5, atol=1e-6)


@pytest.mark.parametrize("rows,heads,width,stride", [(3, 2, 5, 8), (4, 3, 130, 144), (2, 2, 700, 704), (300, 4, 500, 512)])
def test_head_norm_with_padded_heads(rows, heads, width, stride):
    """The padding counts for nothing and comes out as zeros."""
    lib, S, k = _stack()
    g = gen(rows)
    o, gt, w = (torch.randn(*s, heads * stride, generator=g) for s in ((rows,), (rows,), ()))
    O, GT, Wn, res = o.cuda(), gt.cuda(), w.cuda(), torch.full((rows, heads * stride), 9.0).cuda()
    _ok(k.ds41_head_norm_gate(lib.ptr(O), heads * stride, C.byref(S.Proj(GT, heads * stride).args()), lib.ptr(Wn), rows, heads,
                              width, stride, C.c_float(1e-6), lib.ptr(res), heads * stride, 1, lib.stream()))
    v = lambda t: t.view(-1, heads, stride)[..., :width].double()
    want = torch.zeros(rows, heads, stride, dtype=torch.float64)
    want[..., :width] = rms_unit(v(o), 1e-6) * v(w) * torch.sigmoid(v(gt))
    torch.testing.assert_close(res.cpu().double().view(rows, heads, stride), want, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("M,N,K", [(1, 7, 3), (70, 65, 130), (200, 10, 33)])
def test_f32_product_is_true_32_bit(M, N, K):
    lib, S, _ = _stack()
    g = gen(M)
    a, b = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g)
    out = torch.zeros(M, N).cuda()
    S.gemm_f32(a.cuda(), b.cuda(), out, M, N, K, K, K, N)
    torch.testing.assert_close(out.cpu().double(), a.double() @ b.double().T, rtol=1e-5, atol=1e-5)


class AttentionCase:
    """Random cache rows and queries of one request in scattered pages, with chosen keys made to stand out."""

    def __init__(self, heads, dim, rot, vdim, rank, n_keys, rows, dtype, scale=0.2, seed=0, far=None, page=64):
        g = gen(seed)
        r = lambda *s: torch.randn(*s, generator=g).to(dtype).double()
        self.H, self.D, self.Rd, self.V, self.K, self.n, self.rows, self.scale = heads, dim, rot, vdim, rank, n_keys, rows, scale
        self.lat, self.kr, self.q = r(n_keys, rank), r(n_keys, rot), r(rows, heads, dim + rot)
        self.uk, self.uv, self.sink = r(heads, dim, rank) / rank ** 0.5, r(heads, vdim, rank) / rank ** 0.5, r(heads)
        self.uk, self.uv = self.uk.to(dtype).double(), self.uv.to(dtype).double()
        if far is not None:          # one key answers one row's queries far above all others
            row, key = far
            u = torch.sign(self.q[row, :, dim:].sum(0))
            self.q[row, :, dim:] = 3 * u
            self.kr[key] = 4 * u
        self.page, self.dtype = page, dtype
        n_pages = -(-n_keys // page)
        self.order = torch.randperm(n_pages + 3, generator=g)[:n_pages]
        self.n_pages = n_pages + 3

    def want(self):
        n, H = self.n, self.H
        k = torch.cat([torch.einsum("hdc,jc->jhd", self.uk, self.lat), self.kr[:, None].expand(n, H, self.Rd)], -1)
        v = torch.einsum("hvc,jc->jhv", self.uv, self.lat)
        q = torch.zeros(n, H, self.D + self.Rd, dtype=torch.float64)
        q[n - self.rows:] = self.q
        return sink_softmax_attention(q, k, v, self.scale, self.sink)[n - self.rows:]

    def pool(self, kvp, row_len):
        rows = torch.zeros(self.n, row_len, dtype=self.dtype)
        rows[:, :self.K] = self.lat.to(self.dtype)
        rows[:, kvp:kvp + self.Rd] = self.kr.to(self.dtype)
        pool = torch.full((self.n_pages * self.page, row_len), 7.0, dtype=self.dtype)      # other requests' rows
        for i, pg in enumerate(self.order.tolist()):
            part = rows[i * self.page:(i + 1) * self.page]
            pool[pg * self.page:pg * self.page + len(part)] = part
        return pool.cuda(), self.order.int().view(1, -1).contiguous().cuda()


ATTN = [dict(heads=3, dim=20, rot=6, vdim=24, rank=40, n_keys=130, rows=3), dict(heads=18, dim=64, rot=64, vdim=128, rank=128,
        n_keys=300, rows=2), dict(heads=33, dim=16, rot=16, vdim=16, rank=512, n_keys=65, rows=1),
        dict(heads=1, dim=16, rot=2, vdim=16, rank=16, n_keys=64, rows=5)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("splits", [1, 3])
@pytest.mark.parametrize("case", range(len(ATTN)))
def test_absorbed_attention_over_pages(case, splits, dtype):
    """Far keys in other pages, the sink, every split; rows at the end of the sequence."""
    lib, S, k = _stack()
    c = AttentionCase(**ATTN[case], dtype=dtype, far=(0, 1), seed=case)
    kvp, rp = S.ceil_to(c.K, 16), S.ceil_to(c.Rd, 16)
    pool, table = c.pool(kvp, kvp + rp)
    qa = torch.zeros(c.rows, c.H, kvp, dtype=dtype)
    qa[..., :c.K] = torch.einsum("rhd,hdc->rhc", c.q[..., :c.D], c.uk).to(dtype)
    qr = torch.zeros(c.rows, c.H, rp, dtype=dtype)
    qr[..., :c.Rd] = c.q[..., c.D:].to(dtype)
    qa, qr = qa.cuda(), qr.cuda()
    pos = torch.arange(c.n - c.rows, c.n, dtype=torch.int32).cuda()
    slot = torch.zeros(c.rows, dtype=torch.int32).cuda()
    part = torch.zeros(c.rows, splits, c.H, kvp).cuda()
    ml = torch.zeros(c.rows, splits, c.H, 2).cuda()
    out = torch.zeros(c.rows, c.H * kvp, dtype=dtype).cuda()
    a = S.LatentAttendArgs()
    a.q_abs, a.q_rot, a.pool, a.page_table, a.row_pos, a.row_slot, a.part_o, a.part_ml = (
        lib.ptr(t) for t in (qa, qr, pool, table, pos, slot, part, ml))
    a.ld_q_abs, a.ld_q_rot, a.q_rot_stride, a.scale, a.rows, a.heads = c.H * kvp, c.H * rp, rp, c.scale, c.rows, c.H
    a.kv_pad, a.row_len, a.n_splits, a.max_pages, a.page_tokens, a.f32 = kvp, kvp + rp, splits, table.shape[1], c.page, dtype == F32
    _ok(k.ds41_latent_attend(C.byref(a), lib.stream()))
    sink = c.sink.float().cuda()
    _ok(k.ds41_latent_merge(lib.ptr(part), lib.ptr(ml), lib.ptr(sink), splits, c.rows, c.H, kvp, lib.ptr(out), c.H * kvp,
                            int(dtype == F32), lib.stream()))
    o = out.cpu().double().view(c.rows, c.H, kvp)
    assert not o[..., c.K:].any()
    got = torch.einsum("rhc,hvc->rhv", o[..., :c.K], c.uv)
    tol = 2e-5 if dtype == F32 else 0.03
    torch.testing.assert_close(got, c.want(), rtol=tol, atol=tol)


@pytest.mark.parametrize("case", [dict(heads=2, dim=48, rot=16, vdim=48, rank=64, n_keys=129, rows=129),
                                  dict(heads=3, dim=128, rot=64, vdim=128, rank=64, n_keys=700, rows=257),
                                  dict(heads=1, dim=16, rot=16, vdim=16, rank=32, n_keys=1000, rows=64),
                                  dict(heads=2, dim=192, rot=64, vdim=112, rank=64, n_keys=520, rows=300),
                                  dict(heads=2, dim=64, rot=80, vdim=64, rank=64, n_keys=384, rows=256)])
@pytest.mark.parametrize("far", [None, (0, 0), (63, 5)])
def test_prompt_attention_over_expanded_keys(case, far):
    lib, S, k = _stack()
    c = AttentionCase(**case, dtype=BF16, far=far, seed=case["n_keys"])
    dp, rp, vp = S.ceil_to(c.D, 16), S.ceil_to(c.Rd, 16), S.ceil_to(c.V, 16)
    kv = torch.zeros(c.n, c.H * (dp + vp), dtype=BF16)
    keys = torch.einsum("hdc,jc->jhd", c.uk, c.lat).to(BF16)
    vals = torch.einsum("hvc,jc->jhv", c.uv, c.lat).to(BF16)
    kv[:, :c.H * dp].view(c.n, c.H, dp)[..., :c.D] = keys
    kv[:, c.H * dp:].view(c.n, c.H, vp)[..., :c.V] = vals
    rot = torch.zeros(c.n, rp, dtype=BF16)
    rot[:, :c.Rd] = c.kr.to(BF16)
    q = torch.zeros(c.rows, c.H, dp + rp, dtype=BF16)
    q[..., :c.D], q[..., dp:dp + c.Rd] = c.q[..., :c.D].to(BF16), c.q[..., c.D:].to(BF16)
    gate = torch.randn(c.rows, c.H * vp, generator=gen(1))
    q, kv, rot, G, sink = q.cuda(), kv.cuda(), rot.cuda(), gate.cuda(), c.sink.float().cuda()
    out = torch.full((c.rows, c.H * vp), 5.0, dtype=BF16).cuda()
    status = lib.new_status(dev())
    a = S.LatentPrefillArgs()
    a.q, a.kv, a.rot, a.sink, a.out, a.status = (lib.ptr(t) for t in (q, kv, rot, sink, out, status))
    a.gate, a.ld_q, a.ld_kv, a.scale = S.Proj(G, c.H * vp).args(), c.H * (dp + rp), c.H * (dp + vp), c.scale
    a.rows, a.heads, a.dim_pad, a.rot_pad, a.vdim_pad = c.rows, c.H, dp, rp, vp
    a.n_keys, a.pos0, a.ld_out = c.n, c.n - c.rows, c.H * vp
    _ok(k.ds41_latent_prefill(C.byref(a), lib.stream()))
    lib.raise_on_status(status)
    got = out.cpu().double().view(c.rows, c.H, vp)[..., :c.V]
    want = c.want() * torch.sigmoid(gate.double()).view(c.rows, c.H, vp)[..., :c.V]
    torch.testing.assert_close(got, want, rtol=0.03, atol=0.03)


def test_cache_rows_and_queries_are_normed_and_turned():
    lib, S, k = _stack()
    from ds41rt_b200.config import RopeConfig, rope_inv_freq
    rot = dict(base=300.0, dims=10, scaling=dict(factor=3.0, original=40, fast=6.0, slow=0.5))
    rope = RopeConfig(300.0, 3.0, 6.0, 0.5, 40)
    mag = 0.1 * math.log(3.0) + 1.0
    freq = torch.tensor(rope_inv_freq(rope, 10), dtype=F32).cuda()
    g, rows, Q, K, R = gen(3), 6, 24, 40, 10
    x = torch.randn(rows, 24 + 40 + 16, generator=g)
    nq, nk = torch.rand(Q, generator=g) + 0.5, torch.rand(K, generator=g) + 0.5
    pos = torch.tensor([0, 1, 2, 63, 64, 500], dtype=torch.int32)
    slot = torch.tensor([0, 0, 0, 1, 1, -1], dtype=torch.int32)
    table = torch.tensor([[3, -1], [2, 0]], dtype=torch.int32)
    X, cq, pool = x.cuda(), torch.zeros(rows, Q).cuda(), torch.full((4 * 64, 64), 9.0).cuda()
    pin = S.Proj(X, x.shape[1])
    a = S.LatentPostArgs()
    a.dq, a.kv, a.kr = pin.args(), pin.at(24).args(), pin.at(64).args()
    P, SL, T, NQ, NK = pos.cuda(), slot.cuda(), table.cuda(), nq.cuda(), nk.cuda()
    a.dq_norm, a.kv_norm, a.freq, a.cq, a.pool = (lib.ptr(t) for t in (NQ, NK, freq, cq, pool))
    a.page_table, a.row_pos, a.row_slot, a.magnitude, a.eps = lib.ptr(T), lib.ptr(P), lib.ptr(SL), mag, 1e-5
    a.rows, a.q_rank, a.ld_cq, a.kv_rank, a.kv_pad, a.rot_dim, a.row_len = rows, Q, Q, K, 48, R, 64
    a.max_pages, a.page_tokens, a.f32 = 2, 64, 1
    _ok(k.ds41_latent_post(C.byref(a), lib.stream()))
    d = x.double()
    torch.testing.assert_close(cq.cpu().double(), rms_unit(d[:, :Q], 1e-5) * nq, rtol=1e-5, atol=1e-5)
    got, turned = pool.cpu().double(), rotate_pairs(d[:, 64:64 + R], pos, rot)
    lat = rms_unit(d[:, 24:64], 1e-5) * nk
    touched = set()
    for i, at in enumerate((3 * 64, 3 * 64 + 1, 3 * 64 + 2, 2 * 64 + 63, 0)):
        torch.testing.assert_close(got[at, :K], lat[i], rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(got[at, 48:48 + R], turned[i], rtol=1e-4, atol=1e-4)
        touched.add(at)
    assert all((got[i] == 9.0).all() for i in range(256) if i not in touched)
    # queries: two heads of 6 (padded to 8) + 10 (padded to 12)
    q = torch.randn(rows, 2 * 20, generator=g)
    out, Qx = torch.zeros(rows, 40).cuda(), q.cuda()
    _ok(k.ds41_latent_query(C.byref(S.Proj(Qx, 40).args()), lib.ptr(P), lib.ptr(freq), C.c_float(mag), rows, 2, 8, 12, R,
                            lib.ptr(out), 40, 1, lib.stream()))
    want = q.double().view(rows, 2, 20).clone()
    want[..., 8:18] = rotate_pairs(want[..., 8:18], pos, rot)
    torch.testing.assert_close(out.cpu().double().view(rows, 2, 20), want, rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("rows", [5, 300])
def test_latent_norms_of_odd_widths(rows):
    """Both forms of the kernel (one block or one warp per row), widths that end inside a vector."""
    lib, S, k = _stack()
    g, Q, K, R = gen(rows), 1030, 523, 6
    x = torch.randn(2, rows, 1032 + 528 + 8, generator=g)
    nq, nk = torch.rand(Q, generator=g) + 0.5, torch.rand(K, generator=g) + 0.5
    X, NQ, NK, freq = x.cuda(), nq.cuda(), nk.cuda(), torch.tensor([1.0, 0.3, 0.01]).cuda()
    n_pages = -(-rows // 64)
    cq, pool = torch.zeros(rows, 1032).cuda(), torch.zeros(n_pages * 64, 528 + 16).cuda()
    pos, slot = torch.arange(rows, dtype=torch.int32).cuda(), torch.zeros(rows, dtype=torch.int32).cuda()
    table = torch.arange(n_pages - 1, -1, -1, dtype=torch.int32).view(1, -1).contiguous().cuda()
    pin = S.Proj(X, x.shape[2], 2, rows * x.shape[2])
    a = S.LatentPostArgs()
    a.dq, a.kv, a.kr = pin.args(), pin.at(1032).args(), pin.at(1560).args()
    a.dq_norm, a.kv_norm, a.freq, a.cq, a.pool = (lib.ptr(t) for t in (NQ, NK, freq, cq, pool))
    a.page_table, a.row_pos, a.row_slot, a.magnitude, a.eps = lib.ptr(table), lib.ptr(pos), lib.ptr(slot), 1.0, 1e-5
    a.rows, a.q_rank, a.ld_cq, a.kv_rank, a.kv_pad, a.rot_dim, a.row_len = rows, Q, 1032, K, 528, R, 544
    a.max_pages, a.page_tokens, a.f32 = n_pages, 64, 1
    _ok(k.ds41_latent_post(C.byref(a), lib.stream()))
    d = x.double().sum(0)
    got = pool.cpu().double().view(n_pages, 64, 544).flip(0).reshape(-1, 544)[:rows]
    torch.testing.assert_close(cq[:, :Q].cpu().double(), rms_unit(d[:, :Q], 1e-5) * nq, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(got[:, :K], rms_unit(d[:, 1032:1032 + K], 1e-5) * nk, rtol=1e-5, atol=1e-5)
    ang = torch.arange(rows).double()[:, None] * freq.cpu().double()
    u, v = d[:, 1560:1566:2], d[:, 1561:1566:2]
    want = torch.stack([u * ang.cos() - v * ang.sin(), v * ang.cos() + u * ang.sin()], -1).flatten(1)
    torch.testing.assert_close(got[:, 528:534], want, rtol=1e-4, atol=1e-4)
    assert not got[:, 534:].any() and not got[:, K:528].any()


class Recurrence:
    def __init__(self, T, heads, dim, vdim, cap=6.0, seed=0, dtype=F32):
        g = gen(seed)
        r = lambda *s: torch.randn(*s, generator=g)
        self.T, self.H, self.D, self.V, self.cap = T, heads, dim, vdim, cap
        self.q, self.k, self.v = (r(T, heads, n).to(dtype).double() for n in (dim, dim, vdim))
        self.i, self.f = (r(T, heads) * 4).double(), (r(T, heads) * 3 + 2).double()
        self.bi, self.bf = r(heads).double(), r(heads).double()

    def want(self):
        t = lambda x: self.cap * torch.tanh(x / self.cap)
        return mlstm_scan(self.q * self.D ** -0.5, self.k, self.v, t(self.i + self.bi),
                          torch.nn.functional.logsigmoid(t(self.f + self.bf)))

    def run(self, kernel, sizes, dtype, slots=3, slot=1):
        """Feed the sequence in portions of `sizes` through one kernel ("step" / "chunk"; "mix" alternates)."""
        lib, S, k = _stack()
        dp, vp = S.ceil_to(self.D, 16), S.ceil_to(self.V, 16)
        nb = -(-vp // S.STATE_COLS)
        st = [torch.full((slots, self.H) + s, float("nan")).cuda() for s in ((dp, vp), (nb, dp), (nb,))]   # stale states
        pad = lambda x, n: torch.nn.functional.pad(x, (0, n - x.shape[-1])).reshape(self.T, -1)
        q, kk, v = pad(self.q, dp), pad(self.k, dp), pad(self.v, vp)
        x = torch.cat([q, kk, v], 1).to(dtype).cuda()
        gates = torch.cat([self.i, self.f], 1).float().cuda()
        bi, bf = self.bi.float().cuda(), self.bf.float().cuda()
        work = torch.zeros(S.mlstm_chunk_work(self.T, self.H, dp, vp) // 4).cuda()
        outs, at, n_call = [], 0, 0
        while at < self.T:
            n = min(sizes[min(n_call, len(sizes) - 1)], self.T - at)
            px, pg = S.Proj(x[at:], x.shape[1]), S.Proj(gates[at:], gates.shape[1])
            out = torch.full((n, self.H * vp), 3.0).cuda()
            pos = torch.arange(at, at + n, dtype=torch.int32).cuda()
            sl = torch.full((n,), slot, dtype=torch.int32).cuda()
            a = S.MlstmArgs()
            a.q, a.k, a.v = px.args(), px.at(self.H * dp).args(), px.at(2 * self.H * dp).args()
            a.gate_i, a.gate_f, a.bias_i, a.bias_f = pg.args(), pg.at(self.H).args(), lib.ptr(bi), lib.ptr(bf)
            a.row_pos, a.row_slot, a.out, a.work = lib.ptr(pos), lib.ptr(sl), lib.ptr(out), lib.ptr(work)
            a.state_s, a.state_n, a.state_m = (lib.ptr(t) for t in st)
            a.gate_cap, a.q_scale, a.den_eps = self.cap, self.D ** -0.5, 1e-6
            a.rows, a.heads, a.dim_pad, a.vdim_pad, a.slots, a.ld_out = n, self.H, dp, vp, slots, self.H * vp
            which = kernel if kernel != "mix" else ("chunk", "step")[n_call & 1]
            _ok(getattr(k, f"ds41_mlstm_{which}")(C.byref(a), lib.stream()))
            torch.cuda.synchronize()
            outs.append(out.cpu().double().view(n, self.H, vp)[..., :self.V])
            at, n_call = at + n, n_call + 1
        for t in st:                                            # the other slots keep what they held
            assert torch.isnan(t[0]).all() and torch.isnan(t[2]).all() and torch.isfinite(t[1]).all()
        return torch.cat(outs)


@pytest.mark.parametrize("shape", [(2, 24, 40), (1, 16, 16), (3, 64, 96), (1, 100, 32), (1, 200, 64), (1, 400, 16), (1, 600, 48)])
@pytest.mark.parametrize("sizes", [[300], [1], [2, 65, 1, 63]])
def test_recurrence_token_by_token(shape, sizes):
    c = Recurrence(150, *shape, seed=shape[1])
    torch.testing.assert_close(c.run("step", sizes, F32), c.want(), rtol=2e-4, atol=2e-4)


@pytest.mark.parametrize("shape", [(2, 24, 40), (1, 64, 32), (2, 100, 96), (1, 192, 64), (1, 256, 48), (1, 300, 32), (1, 512, 32)])
@pytest.mark.parametrize("kernel,sizes", [("chunk", [300]), ("chunk", [64, 37, 1, 100]), ("mix", [70, 3, 64, 2, 80])])
def test_recurrence_in_chunks(shape, kernel, sizes):
    """Chunk borders, ragged ends, and states handed from one kernel to the other."""
    c = Recurrence(260, *shape, seed=shape[1], dtype=BF16)
    want = c.want()
    got = c.run(kernel, sizes, BF16)
    rel = (got - want).abs() / (want.abs() + want.pow(2).mean(-1, keepdim=True).sqrt() + 1e-2)
    assert torch.isfinite(got).all() and float(rel.max()) < 3e-3


def test_recurrence_keeps_a_token_far_back():
    """Open forget gates and one strong early key: its value is still read hundreds of tokens later."""
    c = Recurrence(400, 1, 32, 32, seed=8, dtype=BF16)
    c.f[:] = 30.0
    c.i[:] = -6.0
    c.i[3] = 5.0
    c.q[-1, 0] = c.k[3, 0]
    want = c.want()
    cos = torch.nn.functional.cosine_similarity(want[-1, 0], c.v[3, 0], dim=0)
    assert float(cos) > 0.99
    torch.testing.assert_close(c.run("chunk", [400], BF16), want, rtol=3e-3, atol=3e-3)
    torch.testing.assert_close(c.run("step", [100, 1], F32), want, rtol=1e-3, atol=1e-3)


def test_bad_arguments_are_refused_on_the_host():
    lib, S, k = _stack()
    assert k.ds41_resid_step(None, lib.stream()) != 0
    a = S.MlstmArgs()
    assert k.ds41_mlstm_step(C.byref(a), lib.stream()) != 0 and k.ds41_mlstm_chunk(C.byref(a), lib.stream()) != 0
    assert k.ds41_latent_prefill(C.byref(S.LatentPrefillArgs()), lib.stream()) != 0
    e = engine("plain", "bf16")
    with pytest.raises(AssertionError):
        e.set_rows([1, 2, 3], [0, 1, 0], [0, 1, 0])               # rows of a request are not adjacent
    with pytest.raises(AssertionError):
        e.set_rows([1, 2], [4, 6], [0, 0])
