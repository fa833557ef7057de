"""Layer-stack models at sizes that resemble a real model's layers, beside a ds41 model of equal size (`bench.py --stack`).

For every preset (random weights, fewer layers than a whole model) and for a ds41 model with the same width, depth,
vocabulary and about the same active weights per token: prompt throughput and decode throughput at several batch sizes, and
the device time of every kernel class with its share of the roofline (measured copy bandwidth or measured bf16 rate,
whichever bounds it).  Decode steps are CUDA-graph replays with on-device token feedback; prompts are eager passes.
"""
from __future__ import annotations

import json
import os
import statistics
from typing import Dict, List, Tuple

import torch

from ..config import ModelConfig, RopeConfig
from ..models import registry
from ..models.stack import state_shapes
from ..runtime.session import DecodeSession
from ..stack_config import StackConfig

FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}


def peaks() -> dict:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            d = json.load(f)
        return {"hbm_gbs": d["hbm_gbs"], "bf16_tflops": d["bf16_tflops"], "source": "measured"}
    return dict(FALLBACK_PEAKS, source="fallback")


def ds41_like(cfg: StackConfig) -> ModelConfig:
    """A ds41 configuration of the same width, depth and vocabulary whose active weights per token are close to cfg's (with
    as many experts, where cfg has mixtures)."""
    W, L = cfg.hidden, cfg.n_layers
    attn = [l.mixer for l in cfg.layers if l.mixer.kind != "mlstm"]
    moe = next((l.mlp for l in cfg.layers if l.mlp is not None and l.mlp.kind == "moe"), None)
    heads = max(m.heads for m in attn)
    q = max(getattr(m, "q_rank", W // 4) for m in attn)
    groups = max(1, heads // 4)
    D, o_lora = 512, 1024 if W >= 4096 else 512
    dense = (q + D) * W + q * heads * D + groups * o_lora * (heads // groups) * D + W * groups * o_lora
    left = stack_layer_weights(cfg) / L - dense
    experts, topk = (moe.experts, moe.top) if moe is not None else (4, 3)
    inter = max(128, int(left / (3 * W * (topk + 1))) // 128 * 128)
    c = ModelConfig(name=f"ds41-like-{cfg.name}", vocab=cfg.vocab, hidden=W, n_layers=L, n_heads=heads, head_dim=D, q_lora=q,
                    o_groups=groups, o_lora=o_lora, window=128, source_layers={0: 1}, compress_ratios=[1] * L,
                    index_layers=tuple(range(0, L, 4)), index_topk=512, candidate_layer=-1, candidate_topk_blocks=0,
                    n_experts=experts, topk=topk, inter=inter, rope_long=RopeConfig(), dspark=None, engram=None, vision=None)
    c.validate()
    return c


def stack_layer_weights(cfg: StackConfig) -> int:
    """Matrix weights of all layers that one token uses."""
    fam = registry.family_of(cfg)
    total = 0
    for l, spec in enumerate(cfg.layers):
        unused = spec.mlp.experts - spec.mlp.top if spec.mlp is not None and spec.mlp.kind == "moe" else 0
        total += sum(s[0] * s[1] for s in fam.layer_shapes(cfg, l).values() if len(s) == 2)
        total -= unused * 3 * cfg.hidden * (spec.mlp.ff if unused else 0)
    return total


def work(cfg: StackConfig, R: int, n_keys: int, first: int, decode: bool, active: int = 0) -> Dict[str, Tuple[float, float]]:
    """Kernel class -> (algorithmic bytes, FLOPs) of one pass of R rows (decode: R requests of n_keys positions each; else
    one request's rows [first, n_keys)), summed over the layers.  `active`: experts that a planned pass uses."""
    W, out = cfg.hidden, {}
    act = 4 if decode else 2           # projections leave as fp32 planes in decode, as bf16 in long passes

    def add(tag, nbytes, flops=0.0):
        b, f = out.get(tag, (0.0, 0.0))
        out[tag] = (b + nbytes, f + flops)

    def gemm(tag, n, k, out_bytes):
        add(tag, 2.0 * n * k + R * (2.0 * k + out_bytes * n), 2.0 * R * n * k)

    def seen(pos, chunk):
        return pos % chunk + 1 if chunk else pos + 1

    for l, spec in enumerate(cfg.layers):
        m = spec.mixer
        chunk = getattr(m, "chunk", 0)
        pairs = R * seen(n_keys - 1, chunk) if decode else sum(seen(p, chunk) for p in range(first, n_keys))
        if m.kind == "grouped_attention":
            H, G = m.heads, m.kv_heads
            cols, row = H * m.dim + G * (m.dim + m.vdim), G * (m.dim + m.vdim)
            back = max(m.taps - 1, 0)
            gemm("gemm_mix_in", cols + (H if m.head_gate else 0), W, act)
            add("attn_post", R * cols * (act + 2.0) + 4.0 * cols * max(m.taps, 1) + (4.0 * R * back * cols if decode else 0))
            if decode:
                add("group_attend", pairs * row * 2.0 + R * H * (m.dim + m.vdim) * 2.0 + (8.0 * R * cols if back else 0),
                    2.0 * pairs * H * (m.dim + m.vdim))
            else:
                low = first - first % chunk if chunk else 0
                add("group_prefill", (n_keys - low) * row * 2.0 + R * H * (m.dim + m.vdim) * 2.0,
                    2.0 * pairs * H * (m.dim + m.vdim))
            gemm("gemm_o", W, H * m.vdim, 4)
        elif m.kind == "latent_attention":
            own = m.kv_from is None
            H, kv = m.heads, m.kv_rank + m.rot_dim
            gemm("gemm_mix_in", m.q_rank + (kv if own else 0) + H * m.vdim + W, W, act)
            add("latent_post", R * ((act + 2.0) * (m.q_rank + (kv if own else 0))))
            gemm("gemm_uq", H * (m.dim + m.rot_dim), m.q_rank, act)
            add("latent_query", R * H * ((m.dim + m.rot_dim) * 6.0 if decode else m.rot_dim * 4.0))
            if decode:
                add("absorb_q", 2.0 * H * m.dim * m.kv_rank + R * H * 2.0 * (m.dim + m.kv_rank), 2.0 * R * H * m.dim * m.kv_rank)
                add("latent_attend", R * n_keys * kv * 2.0 + R * H * kv * 2.0, 2.0 * pairs * H * (kv + m.kv_rank))
                add("latent_merge", R * H * m.kv_rank * 6.0)
                add("values", 2.0 * H * m.vdim * m.kv_rank + R * H * (2.0 * m.kv_rank + 4.0 * m.vdim),
                    2.0 * R * H * m.vdim * m.kv_rank)
                add("gate_mul", R * H * m.vdim * 10.0)
            else:
                if own:
                    add("latent_gather", n_keys * kv * 4.0)
                n = H * (m.dim + m.vdim)
                add("expand_kv", 2.0 * n * m.kv_rank + n_keys * 2.0 * (m.kv_rank + n), 2.0 * n_keys * n * m.kv_rank)
                add("latent_prefill", 2.0 * (n_keys * n + R * H * (m.dim + m.rot_dim + 2 * m.vdim)),
                    2.0 * pairs * H * (m.dim + m.rot_dim + m.vdim))
            gemm("gemm_o", W, H * m.vdim, 4)
        else:
            H, D, V = m.heads, m.dim, m.vdim
            gemm("gemm_mix_in", 2 * H * D + 2 * H * V + W + (2 * H if decode else 0), W, act)
            state = sum(4.0 * a for a in (H * D * V, H * D, H))
            if decode:
                add("mlstm_step", R * (2 * state + 4.0 * H * (2 * D + 2 * V)), R * H * D * V * 6.0)
            else:
                gemm("gemm_gates", 2 * H, W, 4)
                add("mlstm_chunk", 2 * state + R * (2.0 * H * (2 * D + V) + 4.0 * H * V),
                    R * H * (2.0 * 64 * (D + V) + 4.0 * D * V))
            add("head_norm_gate", R * H * V * (6.0 + act))
            gemm("gemm_o", W, H * V, 4)
        ml = spec.mlp
        gate = act if cfg.residual_gate else 0
        # result, gate and stream in, stream and next input out
        add("resid_step", R * W * (4.0 + gate + 4 + 4 + 2))
        if ml is not None and ml.kind == "dense":
            gemm("gemm_up", ml.ff + W, W, act)
            add("polynorm", R * ml.ff * (act + 2.0))
            gemm("gemm_down", W, ml.ff, 4)
            add("resid_step", R * W * (4.0 + gate + 4 + 4 + 2))
        elif ml is not None:
            routes = R * ml.top
            gemm("gemm_router", ml.experts, W, 4)
            add("route", R * ml.experts * 4.0 + routes * 8.0)
            if decode and active:
                add("gemm_fc1", active * 4.0 * ml.ff * W + R * 2.0 * W + routes * 2.0 * ml.ff, routes * 4.0 * ml.ff * W)
                add("gemm_fc2", active * 2.0 * ml.ff * W + routes * (2.0 * ml.ff + 4.0 * W), routes * 2.0 * ml.ff * W)
            else:
                used = min(ml.experts, routes)
                add("ep_moe", used * 6.0 * ml.ff * W + R * 2.0 * W + routes * 2.0 * (2 * W + 2 * ml.ff), routes * 6.0 * ml.ff * W)
            add("resid_step", R * W * (ml.top * (4.0 if decode and active else 2.0) + gate + 4 + 4 + 2))
        if cfg.token_side:
            gemm("gemm_side_gate", cfg.token_side, W, 4)
            add("side_act", R * cfg.token_side * 8.0)
            gemm("gemm_side_proj", W, cfg.token_side, 4)
            add("resid_step", R * W * (4.0 + 4 + 4 + 2))
        if cfg.depth_average:          # reads every kept stream and writes the sum
            add("resid_step", R * W * (4.0 * (l + 1) + 4))
    add("resid_step", R * W * 8.0)
    heads = R if decode else 1
    add("gemm_head", 2.0 * cfg.vocab * W + 4.0 * heads * cfg.vocab, 2.0 * heads * cfg.vocab * W)
    add("argmax_rows", 4.0 * heads * cfg.vocab)
    return out


def _timed(fn, reps: int) -> float:
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(reps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / reps


def _classes(e, run) -> Dict[str, List[float]]:
    """tag -> [launches, total us] of one eager pass with an event pair around every launch."""
    e.timeline = []
    run()
    torch.cuda.synchronize()
    acc: Dict[str, List[float]] = {}
    for tag, a, b in e.timeline:
        x = acc.setdefault(tag, [0, 0.0])
        x[0] += 1
        x[1] += a.elapsed_time(b) * 1e3
    e.timeline = None
    return acc


def bench_engine(e, prompt_len: int, chunk: int, batches, steps: int, warmup: int, context: int, work_of=None) -> dict:
    pk = peaks()
    g = torch.Generator().manual_seed(1234)
    prompt = torch.randint(3, e.cfg.vocab - 3, (prompt_len,), generator=g).tolist()

    def table(acc, w):
        rows = {}
        for tag, (n, us) in sorted(acc.items(), key=lambda kv: -kv[1][1]):
            row = {"launches": n, "us_each": round(us / n, 2)}
            if w is not None and tag in w:
                nbytes, flops = w[tag]
                t_mem, t_mma = nbytes / pk["hbm_gbs"] / 1e3, flops / pk["bf16_tflops"] / 1e6
                row["bound"] = "hbm" if t_mem >= t_mma else "tensor"
                row["roofline"] = round(max(t_mem, t_mma) / us, 3)
            rows[tag] = row
        return rows

    for _ in range(max(3, warmup)):
        e.prefill(0, prompt, chunk=chunk)
    ms = statistics.median(_timed(lambda: e.prefill(0, prompt, chunk=chunk), 1) for _ in range(max(3, steps // 8)))
    # kernel classes of the last pass of the prompt
    first = (prompt_len - 1) // chunk * chunk
    n = prompt_len - first

    def last_pass():
        e.set_rows(prompt[first:], list(range(first, prompt_len)), [0] * n)
        e.forward_rows(n, head=True, head_row=n - 1)

    last_pass()
    rep = {"prefill": {"prompt": prompt_len, "chunk": chunk, "tok_s": round(prompt_len / ms * 1e3, 1), "ms": round(ms, 3),
                       "last_pass_kernels": table(_classes(e, last_pass),
                                                  work_of(n, prompt_len, first, False) if work_of else None)}}
    e.check_status("prompt passes")
    e.cache.release(0)
    rep["decode"] = []
    for B in batches:
        for s in range(B):
            assert e.cache.ensure(s, context + 4 * (steps + warmup) + 64)
        rows = ([(5 + 37 * s) % e.cfg.vocab for s in range(B)], [context] * B, list(range(B)))
        ses = DecodeSession(e)
        e.set_rows(*rows)
        ses.graph(B, feedback=True)
        ses.run_device_loop(B, max(3, warmup))
        ms = statistics.median(_timed(lambda: ses.run_device_loop(B, steps), 1) / steps for _ in range(3))
        launches = ses.launches_per_graph[(B, True)]
        # a kernel class alone: the same graph with every other launch left out
        e.set_rows(*rows)
        counts = {t: c for t, (c, _) in _classes(e, lambda: e.forward_rows(B)).items()}
        active = int(e.n_active) if work_of and "gemm_fc1" in counts else 0      # what the last layer's routes left
        acc = {}
        for tag, c in counts.items():
            e.only = {tag}
            alone = DecodeSession(e)
            e.set_rows(*rows)
            alone.graph(B)
            alone.graph(B).replay()
            acc[tag] = [c, _timed(lambda: alone.graph(B).replay(), 10) * 1e3]
            e.only = None
        rep["decode"].append({"batch": B, "context": context, "ms_per_step": round(ms, 4), "tok_s": round(B / ms * 1e3, 1),
                              "launches": launches,
                              "kernels": table(acc, work_of(B, context + 1, 0, True, active) if work_of else None)})
        e.check_status("decode")
        for s in range(B):
            e.cache.release(s)
    return rep


def run(names: List[str], dev, steps: int, warmup: int, prompt: int, chunk: int, layers: int, context: int,
        batches=(1, 8, 32)) -> dict:
    out = {"peaks": peaks(), "models": {}}
    for name in names:
        fam, cfg = registry.preset(name, layers or {"1b": 16, "7b": 8}.get(name.split("-")[-1], 0))
        like = ds41_like(cfg)
        max_ctx = max(prompt, context + 4 * (steps + warmup) + 64) // 64 * 64 + 128
        for family, c in ((fam, cfg), (registry.FAMILIES["ds41"], like)):
            kw = {} if family is fam else {"expert_dtype": "bf16"}
            w = family.random_weights(c, dev, seed=0, **kw)
            e = family.engine(c, w, max_rows=chunk, slots=max(batches), max_ctx=max_ctx)
            rep = bench_engine(e, prompt, chunk, batches, steps, warmup, context,
                               (lambda *a: work(cfg, *a)) if family is fam else None)
            rep.update(layers=c.n_layers, hidden=c.hidden, vocab=c.vocab, weights_gb=round(w.nbytes() / 1e9, 2),
                       layer_weights_per_token_m=round(stack_layer_weights(cfg) / c.n_layers / 1e6, 1) if family is fam
                       else ds41_active(c))
            if family is fam:
                rep["state_mb_per_request"] = round(sum(4 * _prod(s) for l in c.state_layers()
                                                        for s in state_shapes(c.layers[l].mixer)) / 1e6, 2)
            out["models"][c.name] = rep
            del e, w
            torch.cuda.empty_cache()
    return out


def _prod(s):
    n = 1
    for x in s:
        n *= x
    return n


def ds41_active(c: ModelConfig) -> float:
    """Millions of active matrix weights per layer and token (dense part, shared expert, topk experts)."""
    dense = (c.q_lora + c.head_dim) * c.hidden + c.q_lora * c.n_heads * c.head_dim + \
        c.o_groups * c.o_lora * c.heads_per_group * c.head_dim + c.hidden * c.o_groups * c.o_lora
    return round((dense + 3 * c.hidden * c.inter * (c.topk + 1)) / 1e6, 1)
