"""Genesun on the host: configuration, tensor catalog, registry, memory plan, cache bookkeeping, and the oracle's own
self-checks (a chunked form of the recurrence, a mistake that must show)."""
import copy
import json

import pytest
import torch

from ds41rt_b200.loader.safetensors_io import SafetensorsError, write_safetensors
from ds41rt_b200.loader.stack import StackCheckpoint
from ds41rt_b200.models import genesun, registry
from ds41rt_b200.models.stack import StackCache, latent_row_len
from ds41rt_b200.stack_config import ConfigError
from genesun_oracle import (MODELS, GenesunOracle, make_weights, mlstm_scan, position_error, sink_softmax_attention,
                            yarn_frequencies)


@pytest.mark.parametrize("name", list(MODELS))
def test_tensor_catalog_is_what_a_model_holds(name):
    cfg = genesun.parse(MODELS[name], name)
    assert genesun.tensor_shapes(cfg) == {k: tuple(v.shape) for k, v in make_weights(MODELS[name]).items()}


def test_configuration_is_read_strictly():
    doc = MODELS["odd"]
    cfg = genesun.parse(doc)
    assert [l.mixer.kind for l in cfg.layers] == ["latent_attention", "mlstm", "latent_attention", "latent_attention"]
    assert cfg.cache_layers() == [0] and cfg.state_layers() == [1] and cfg.source_of(3) == 0 and cfg.source_of(1) is None
    assert cfg.layers[2].mlp is None and cfg.layers[1].mlp.ff == 60 and cfg.norm_eps == 1e-6

    def broken(change):
        d = copy.deepcopy(doc)
        change(d)
        with pytest.raises(ConfigError):
            genesun.parse(d)

    broken(lambda d: d.update(extra=1))
    broken(lambda d: d["layers"][0]["mixer"].pop("scale"))
    broken(lambda d: d["layers"][1].update(type="mamba"))
    broken(lambda d: d["layers"][3]["mixer"].update(kv_from=2))             # a layer without rows of its own
    broken(lambda d: d["layers"][3]["mixer"].update(kv_from=1))
    broken(lambda d: d["layers"][3]["mixer"].update(kv_rank=48))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=8))
    broken(lambda d: d["layers"][0]["mlp"].update(kind="moe"))


def test_rotation_frequencies_agree_with_the_plain_statement():
    from ds41rt_b200.config import rope_inv_freq
    for name in MODELS:
        for spec, d in zip(genesun.parse(MODELS[name]).layers, MODELS[name]["layers"]):
            if d["type"] == "latent_attention":
                freq, mag = yarn_frequencies(d["mixer"]["rot"])
                assert rope_inv_freq(spec.mixer.rope, spec.mixer.rot_dim) == pytest.approx(freq, rel=1e-12)
                assert spec.mixer.magnitude == pytest.approx(mag, rel=1e-12)
    # both ends of the ramp at the same place, and past the last pair
    for sc in (dict(factor=4.0, original=64, fast=1.0, slow=1.0), dict(factor=4.0, original=1 << 20, fast=2.0, slow=1.0)):
        rot = dict(base=100.0, dims=8, scaling=sc)
        assert rope_inv_freq(genesun._rope(rot, 8, "rot"), 8) == pytest.approx(yarn_frequencies(rot)[0], rel=1e-12)


def test_checkpoint_and_registry(tmp_path):
    doc, w = MODELS["plain"], {k: v.to(torch.bfloat16) for k, v in make_weights(MODELS["plain"], 3).items()}
    (tmp_path / "config.json").write_text(json.dumps(doc))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    fam, cfg = registry.config_from_file(str(tmp_path))
    assert fam.name == "genesun" and registry.family_of(cfg) is fam
    ck = StackCheckpoint(str(tmp_path), genesun.tensor_shapes(cfg))
    assert all(torch.equal(ck.read(n), t) for n, t in w.items())
    sw = genesun.build_weights(cfg, ck.read, "cpu", "f32")
    assert torch.equal(sw.head.w[:, :cfg.hidden], w["head"].float()) and sw.nbytes() > 0
    for change in (lambda d: d.pop("l0.dwa"), lambda d: d.update(extra=torch.zeros(1)),
                   lambda d: d.update({"l0.dwa": torch.zeros(3)})):
        bad = dict(w)
        change(bad)
        write_safetensors(str(tmp_path / "model.safetensors"), bad)
        with pytest.raises(SafetensorsError):
            StackCheckpoint(str(tmp_path), genesun.tensor_shapes(cfg))
    with pytest.raises(registry.UnsupportedDtype):
        registry.FAMILIES["ds41"].random_weights(registry.preset("tiny")[1], "cpu", dtype="f32")
    assert registry.preset("flash", 3)[1].n_layers == 3 and registry.preset("genesun-tiny")[0].name == "genesun"
    with pytest.raises(ValueError):
        registry.preset("nothing")


def test_memory_plan_counts_rows_and_states():
    from ds41rt_b200.runtime.memory import plan_pool, stack_page_bytes, stack_state_bytes
    cfg = genesun.parse(MODELS["odd"])
    row = latent_row_len(cfg.layers[0].mixer)[1]
    assert row == 48 + 16 and stack_page_bytes(cfg, 64) == 64 * row * 2
    assert stack_state_bytes(cfg) == 4 * (3 * 32 * 48 + 3 * 2 * 32 + 3 * 2)
    plan = plan_pool(cfg, n_layers=4, slots=4, max_context=1000, free_bytes=8 << 30, retained=10)
    assert plan.pages == plan.pages_wanted and plan.ring_bytes == 14 * stack_state_bytes(cfg)


def test_snapshots_share_full_pages_and_copy_the_rest():
    cfg = genesun.parse(MODELS["odd"])
    c = StackCache(cfg, 2, 512, torch.device("cpu"), torch.float32, n_pages=8)
    assert c.ensure(0, 150)
    pages = c.pages_of(0)
    for t in c.pools.values():
        t.copy_(torch.arange(t.shape[0])[:, None].expand_as(t))
    for st in c.states.values():
        for t in st:
            t[0] = 5.0
    snap = c.snapshot(0, 150)
    assert snap.pages == pages[:2] and snap.partial[0].shape[0] == 22 and snap.nbytes() > 0
    c.release(0)
    for st in c.states.values():
        for t in st:
            t.zero_()
    assert c.restore(1, snap) and c.pages_of(1)[:2] == pages[:2]
    at = c.pages_of(1)[2] * 64
    assert torch.equal(c.pools[0][at:at + 22, 0], torch.arange(pages[2] * 64, pages[2] * 64 + 22).float())
    assert all((t[1] == 5.0).all() and not t[0].any() for t in c.states[1])
    assert not c.restore_prefix(0, snap, 128)
    c.release(1)
    c.drop_snapshot(snap)
    assert c.free_pages == 8


def test_oracle_recurrence_in_its_chunked_form():
    """The chunk algebra of the tensor-core kernel, in plain form, against the token-by-token scan."""
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    T, D, V, L = 100, 8, 6, 16
    q, k, v, i, f = r(T, 1, D), r(T, 1, D), r(T, 1, V), 3 * r(T, 1), -r(T, 1).abs()
    want = mlstm_scan(q, k, v, i, f)
    S, n, m0, out = torch.zeros(D, V, dtype=torch.float64), torch.zeros(D, dtype=torch.float64), torch.tensor(0.0), []
    for c in range(0, T, L):
        qc, kc, vc, ic, fc = q[c:c + L, 0], k[c:c + L, 0], v[c:c + L, 0], i[c:c + L, 0], f[c:c + L, 0]
        F = fc.cumsum(0)
        m = F + torch.maximum(torch.cummax(ic - F, 0).values, m0)
        dec = (F[:, None] - F[None] + ic[None] - m[:, None]).exp().tril()
        P = (qc @ kc.T) * dec
        inter = (F + m0 - m).exp()
        num = inter[:, None] * (qc @ S) + P @ vc
        den = torch.maximum((inter * (qc @ n) + P.sum(1)).abs(), (-m).exp()) + 1e-6
        out.append(num / den[:, None])
        w = (F[-1] - F + ic - m[-1]).exp()
        keep = (F[-1] + m0 - m[-1]).exp()
        S, n, m0 = keep * S + (w[:, None] * kc).T @ vc, keep * n + w @ kc, m[-1]
    torch.testing.assert_close(torch.cat(out), want[:, 0], rtol=1e-9, atol=1e-12)


def test_a_planted_mistake_shows_in_the_logits():
    """Each mechanism left out of the oracle moves the logits hundreds of times beyond the 32-bit bounds."""
    doc, w = MODELS["odd"], make_weights(MODELS["odd"], 1)
    toks = torch.randint(0, doc["vocab"], (60,), generator=torch.Generator().manual_seed(2)).tolist()
    want = GenesunOracle(doc, w).forward(toks)[0]

    def moved(change_doc=lambda d: None, change_w=lambda x: None):
        d, x = copy.deepcopy(doc), dict(w)
        change_doc(d)
        change_w(x)
        return float(position_error(GenesunOracle(d, x).forward(toks)[0], want).median())

    assert moved() == 0.0
    assert moved(change_w=lambda x: x.update({"l0.mix.sink": torch.full((3,), -100.0)})) > 5e-3
    assert moved(change_w=lambda x: x.update({"l2.dwa": torch.tensor([0.0, 0.0, 0.0, 1.0])})) > 5e-3
    assert moved(change_w=lambda x: x.update({"l0.mlp.act": w["l0.mlp.act"] * torch.tensor([1.0, 1.0, 0.0, 1.0])})) > 5e-3
    assert moved(change_w=lambda x: x.update({"l1.rg1.b": torch.zeros(90)})) > 5e-3
    assert moved(lambda d: d["layers"][0]["mixer"]["rot"].pop("scaling")) > 5e-3
    assert moved(lambda d: d["layers"][1]["mixer"].update(gate_cap=70.0)) > 5e-3
    assert moved(lambda d: d["layers"][3]["mixer"].update(scale=0.1)) > 5e-3


def test_oracle_attention_counts_the_sink_once():
    q = torch.zeros(3, 1, 4, dtype=torch.float64)
    v = torch.ones(3, 1, 2, dtype=torch.float64)
    out = sink_softmax_attention(q, q, v, 1.0, torch.zeros(1, dtype=torch.float64))
    assert out[:, 0, 0].tolist() == pytest.approx([1 / 2, 2 / 3, 3 / 4])
