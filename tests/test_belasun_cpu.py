"""Belasun on the host: configuration, tensor catalog, registry, command line, memory plan, snapshots, and the oracle's own
self-checks (other forms of the same equations, mistakes that must show)."""
import copy
import json
import math
import subprocess
import sys

import pytest
import torch

from belasun_oracle import (BANDS, MODELS, BelasunOracle, chunk_visible, expert, frequencies, make_weights, masked_attention,
                            position_error, rotate_halves, route, short_conv)
from ds41rt_b200.loader.safetensors_io import SafetensorsError, write_safetensors
from ds41rt_b200.loader.stack import StackCheckpoint
from ds41rt_b200.models import belasun, registry
from ds41rt_b200.models.stack import StackCache, cache_row_len, state_shapes
from ds41rt_b200.stack_config import ConfigError


@pytest.mark.parametrize("name", list(MODELS))
def test_tensor_catalog_is_what_a_model_holds(name):
    cfg = belasun.parse(MODELS[name], name)
    assert belasun.tensor_shapes(cfg) == {k: tuple(v.shape) for k, v in make_weights(MODELS[name]).items()}


def test_configuration_is_read_strictly():
    doc = MODELS["odd"]
    cfg = belasun.parse(doc)
    assert [(l.mixer.heads, l.mixer.kv_heads, l.mixer.chunk, l.mixer.taps, l.mixer.rot_dim) for l in cfg.layers] == \
        [(6, 2, 37, 3, 12), (3, 3, 100, 5, 12), (5, 1, 16, 2, 20)]
    assert cfg.layers[1].mlp is None and (cfg.layers[2].mlp.experts, cfg.layers[2].mlp.top, cfg.layers[2].mlp.ff) == (7, 3, 20)
    assert cfg.layers[0].mlp.limit == 1.5 and cfg.norm_eps == 1e-5 and cfg.token_side == 10 and cfg.logit_softcap == 20.0
    assert cfg.cache_layers() == [0, 1, 2] and cfg.state_layers() == [0, 1, 2] and cfg.norm_kind == 1
    assert cfg.layers[0].mixer.rope.bands == (1.0, 5.0) and cfg.layers[1].mixer.rope.bands is None

    def broken(change):
        d = copy.deepcopy(doc)
        change(d)
        with pytest.raises(ConfigError):
            belasun.parse(d)

    broken(lambda d: d.update(extra=1))
    broken(lambda d: d["layers"][0]["mixer"].pop("scale"))
    broken(lambda d: d["layers"][0]["mixer"].update(window=3))
    broken(lambda d: d["layers"][0].update(type="mlstm"))
    broken(lambda d: d["layers"][0]["mixer"].update(kv_heads=4))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=22))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7))
    broken(lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("low"))
    broken(lambda d: d["layers"][0]["mixer"]["mask"].update(size=0))
    broken(lambda d: d["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=6))
    broken(lambda d: d["layers"][0]["mlp"]["expert"].pop("limit"))


def test_rotation_frequencies_agree_with_the_plain_statement():
    from ds41rt_b200.config import rope_inv_freq
    rots = [l["mixer"]["rot"] for m in MODELS.values() for l in m["layers"]]
    rots += [dict(base=100.0, dims=64, scaling=dict(factor=4.0, low=a, high=b, original=o))
             for a, b, o in ((1.0, 4.0, 100), (2.0, 3.0, 40), (0.5, 64.0, 1000))]
    for rot in rots:
        dims, rope = belasun._rope(rot, "rot")
        assert rope_inv_freq(rope, dims) == pytest.approx(frequencies(rot), rel=1e-12)
    kept, slowed = frequencies(dict(base=100.0, dims=64)), frequencies(rots[-3])
    ratio = [a / b for a, b in zip(kept, slowed)]
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(4.0) and any(1.01 < r < 3.99 for r in ratio)     # all three bands


def test_checkpoint_and_registry(tmp_path):
    doc, w = MODELS["plain"], {k: v.to(torch.bfloat16) for k, v in make_weights(MODELS["plain"], 3).items()}
    (tmp_path / "config.json").write_text(json.dumps(doc))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    fam, cfg = registry.config_from_file(str(tmp_path))
    assert fam.name == "belasun" and registry.family_of(cfg) is fam
    ck = StackCheckpoint(str(tmp_path), fam.tensor_shapes(cfg))
    assert all(torch.equal(ck.read(n), t) for n, t in w.items())
    sw = belasun.build_weights(cfg, ck.read, "cpu", "f32")
    assert torch.equal(sw.head.w[:, :cfg.hidden], w["embed"].float()) and torch.equal(sw.side_embed, w["side.embed"])
    assert torch.equal(sw.layers[0].mlp.w13[0, :16, :64], w["l0.mlp.e0.gate"].float())
    tied = belasun.build_weights(cfg, ck.read, "cpu", "bf16")
    assert tied.head is tied.embed and tied.nbytes() < sw.nbytes()
    for change in (lambda d: d.pop("l0.side.norm"), lambda d: d.update(extra=torch.zeros(1)),
                   lambda d: d.update({"l0.mix.q.conv": torch.zeros(16, 3)})):
        bad = dict(w)
        change(bad)
        write_safetensors(str(tmp_path / "model.safetensors"), bad)
        with pytest.raises(SafetensorsError):
            StackCheckpoint(str(tmp_path), fam.tensor_shapes(cfg))
    for name in belasun.PRESETS:
        fam, cfg = registry.preset(name, 2)
        assert fam.name == "belasun" and cfg.n_layers == 2 and cfg.max_context > 8192


@pytest.mark.parametrize("command", ["info", "inspect-model"])
def test_command_line_describes_a_preset(command):
    out = subprocess.run([sys.executable, "-m", "ds41rt_b200", command, "--model", "belasun-1b", "--layers", "2"],
                         capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr[-500:]
    doc = json.loads(out.stdout)
    assert doc["family"] == "belasun" and doc.get("checkpoint_tensors", doc.get("tensors")) == 3 + 2 * (14 + 3 + 32 * 3)


def test_memory_plan_counts_rows_and_convolution_inputs():
    from ds41rt_b200.runtime.memory import plan_pool, stack_page_bytes, stack_state_bytes
    cfg = belasun.parse(MODELS["odd"])
    rows = [2 * (32 + 32), 3 * (16 + 48), 1 * (32 + 32)]
    assert [cache_row_len(l.mixer) for l in cfg.layers] == rows and stack_page_bytes(cfg, 64) == 64 * 2 * sum(rows)
    cols = [6 * 32 + rows[0], 3 * 16 + rows[1], 5 * 32 + rows[2]]
    assert stack_state_bytes(cfg) == 4 * (2 * cols[0] + 4 * cols[1] + 1 * cols[2])
    plan = plan_pool(cfg, n_layers=3, slots=4, max_context=1000, free_bytes=8 << 30, retained=10)
    assert plan.pages == plan.pages_wanted and plan.ring_bytes == 14 * stack_state_bytes(cfg)
    one_tap = belasun.parse(MODELS["plain"])
    assert one_tap.state_layers() == [0, 2] and state_shapes(one_tap.layers[0].mixer) == ((3, 48),)


def test_snapshots_carry_the_convolution_inputs():
    cfg = belasun.parse(MODELS["odd"])
    c = StackCache(cfg, 2, 512, torch.device("cpu"), torch.float32, n_pages=8)
    assert c.ensure(0, 70)
    for st in c.states.values():
        st[0][0] = 3.0
    snap = c.snapshot(0, 70)
    c.release(0)
    for st in c.states.values():
        st[0].zero_()
    assert c.restore(1, snap) and all((st[0][1] == 3.0).all() and not st[0][0].any() for st in c.states.values())
    assert not c.restore_prefix(0, snap, 64)
    c.release(1)
    c.drop_snapshot(snap)
    assert c.free_pages == 8


# ---------------------------------------------------------------------------------------------------- the oracle itself
def r(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_oracle_convolution_is_the_library_one():
    u, w = r(30, 7), r(7, 4, seed=1)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(u.T, (3, 0))[None], w[:, None], groups=7)[0].T
    torch.testing.assert_close(short_conv(u, w), want)


def test_oracle_attention_in_its_chunks():
    """Chunk by chunk with a plain causal mask is the masked attention of the whole sequence."""
    q, k, v = r(50, 6, 8), r(50, 2, 8, seed=1), r(50, 2, 5, seed=2)
    want = masked_attention(q, k, v, 0.7, chunk_visible(50, 16))
    parts = [masked_attention(q[a:a + 16], k[a:a + 16], v[a:a + 16], 0.7, chunk_visible(min(16, 50 - a), None))
             for a in range(0, 50, 16)]
    torch.testing.assert_close(torch.cat(parts), want)
    seen = chunk_visible(40, 16)
    assert seen[16].nonzero().tolist() == [[16]] and seen[15].sum() == 16 and not seen[31, 32] and seen[39].sum() == 8


def test_oracle_rotation_depends_on_distance_alone():
    rot = dict(base=30.0, dims=8, scaling=BANDS)
    q, k = r(1, 1, 12), r(1, 1, 12, seed=1)

    def score(i, j):
        a, b = rotate_halves(q, torch.tensor([i]), rot), rotate_halves(k, torch.tensor([j]), rot)
        assert torch.equal(a[..., 8:], q[..., 8:])
        return float((a * b).sum())

    assert score(9, 4) == pytest.approx(score(109, 104)) and abs(score(9, 4) - score(9, 5)) > 1e-3
    # value 0 turns with value 4: a quarter turn moves one into the other
    x = torch.zeros(1, 1, 12, dtype=torch.float64)
    x[..., 0] = 1.0
    y = rotate_halves(x, torch.tensor([1]), dict(base=1.0, dims=8))
    assert y[0, 0, 0] == pytest.approx(math.cos(1)) and y[0, 0, 4] == pytest.approx(math.sin(1)) and not y[0, 0, 1:4].any()


def test_oracle_router_and_expert():
    w = {"router": torch.eye(4, dtype=torch.float64), "router.b": torch.tensor([0.0, 0.0, 3.0, 0.0], dtype=torch.float64)}
    ids, wt = route(torch.tensor([[1.0, 2.0, 0.5, -1.0]], dtype=torch.float64), w, "", 2)
    assert ids.tolist() == [[2, 1]] and wt[0, 0] == pytest.approx(1 / (1 + math.exp(-1.5)))
    one = {n: torch.ones(1, 1, dtype=torch.float64) for n in ("gate", "up", "down")}
    h = torch.tensor([[5.0], [-5.0]], dtype=torch.float64)
    got = expert(h, one, "", 2.0)[:, 0]
    assert got[0] == pytest.approx(2 / (1 + math.exp(-1.702 * 2)) * 3)              # both parts cut at the limit
    assert got[1] == pytest.approx(-5 / (1 + math.exp(1.702 * 5)) * -1)             # the gate has no lower limit


def test_a_planted_mistake_shows_in_the_logits():
    """Each mechanism left out of the oracle moves the logits hundreds of times beyond the 32-bit bounds."""
    doc, w = MODELS["odd"], make_weights(MODELS["odd"], 1)
    toks = torch.randint(0, doc["vocab"], (60,), generator=torch.Generator().manual_seed(2)).tolist()
    want = BelasunOracle(doc, w).forward(toks)[0]

    def moved(change_doc=lambda d: None, change_w=lambda x: None):
        d, x = copy.deepcopy(doc), dict(w)
        change_doc(d)
        change_w(x)
        return position_error(BelasunOracle(d, x).forward(toks)[0], want)

    assert float(moved().max()) == 0.0

    def shows(*a, rows=slice(None)):
        assert float(moved(*a)[rows].median()) > 5e-3

    mixer0 = lambda d: d["layers"][0]["mixer"]
    shows(lambda d: mixer0(d)["rot"].pop("scaling"), rows=slice(10, 37))
    shows(lambda d: mixer0(d)["mask"].update(size=36), rows=slice(36, 60))
    shows(lambda d: mixer0(d)["mask"].update(size=38), rows=slice(37, 60))
    shows(lambda d: mixer0(d).update(scale=0.2))
    shows(lambda d: mixer0(d)["rot"].update(dims=20))
    shows(lambda d: d["layers"][0]["mlp"]["expert"].update(limit=1.4))
    shows(lambda d: d["layers"][2]["mlp"]["router"].update(top=2))
    shows(lambda d: d["norm"].update(eps=3e-2))
    shows(lambda d: d.update(logit_softcap=25.0))
    for name, t in (("l0.mix.q.conv", w["l0.mix.q.conv"] * torch.tensor([0.0, 1.0, 1.0])),
                    ("l1.mix.v.conv", w["l1.mix.v.conv"] * torch.tensor([0.0, 1.0, 1.0, 1.0, 1.0])),
                    ("l0.mix.k.norm", torch.ones(40)), ("l1.mix.g", torch.zeros(3, 90)),
                    ("l0.mlp.router.b", torch.zeros(5)), ("side.embed", w["side.embed"].roll(1, 1)),
                    ("l2.side.norm", torch.ones(90))):
        shows(lambda d: None, lambda x, name=name, t=t: x.update({name: t}))


def test_steady_models_route_with_a_margin():
    for name, doc in MODELS.items():
        w = make_weights(doc, 1, steady=True)
        toks = torch.randint(0, doc["vocab"], (80,), generator=torch.Generator().manual_seed(3)).tolist()
        used, o = set(), BelasunOracle(doc, w)
        _, after = o.forward(toks)
        code = max(d["mlp"]["router"]["experts"] for d in doc["layers"] if d["mlp"])
        for x in after:
            if code > 1:
                # nothing but the per-layer token input writes to the code, and that not at all
                torch.testing.assert_close(x[:, :code], o.w["embed"][toks][:, :code])
                used |= set(x[:, :code].argmax(-1).tolist())
        assert code == 1 or len(used) > code // 2
