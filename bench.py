#!/usr/bin/env python
"""bench.py — decode tokens/s (bf16, batch 1) of the B200 decode engine, with roofline and CPU baseline.

    python bench.py [--gpus N] [--steps K] [--warmup W] [--model Qwen2.5-0.5B] [--impl ours|reference]
    python -m torch.distributed.run --nnodes=1 --nproc-per-node N --master-addr 127.0.0.1 --master-port P \
        bench.py --gpus N --steps K --warmup W

A "step" is ONE 128-token greedy decode of one sequence (Qwen2.5-0.5B bf16, batch 1,
128-token decode) continuing a 16-token prompt: rewind to position 16, run 128 engine steps on the device.
`value` = decoded tokens / second with everything resident in HBM (CUDA events on the launching stream).
`e2e`   = the same through the public API with HOST buffers: DecodeEngine.generate_sync(prompt ids on the host) —
          H2D of the prompt, cache reset, 16-token prefill, 127 decode steps, D2H of the 128 ids, all inside the clock.
Synthetic seeded weights of the real shape (no checkpoints offline); weights (0.99 GB) ≫ L2 (126 MB), so every token
re-streams them from HBM — no explicit L2 flush is needed and none is done.
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

PROMPT_LEN = 16
NEW_TOKENS = 128


def measured_peaks():
    p = ROOT / "MEASURED_PEAKS.json"
    if p.exists():
        try:
            d = json.loads(p.read_text())
            return float(d["hbm_gbs"]), "measured (MEASURED_PEAKS.json hbm_gbs)"
        except Exception:
            pass
    return 6650.0, "fallback (B200_PROFILING.md 6.65 TB/s)"


class ClockSampler:
    """nvidia-smi clocks/throttle reasons sampled DURING the timed region (one streaming `nvidia-smi -lms 100`)."""
    Q = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,clocks_event_reasons.hw_slowdown,"
         "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
         "clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu_index: int):
        self.idx = gpu_index
        self.rows = []
        self._p = None

    def __enter__(self):
        try:
            self._p = subprocess.Popen(["nvidia-smi", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits", "-i",
                                        str(self.idx), "-lms", "100"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL,
                                       text=True)
            time.sleep(0.35)  # first sample before the timed region starts
        except Exception:
            self._p = None
        return self

    def __exit__(self, *a):
        if self._p is None:
            return
        time.sleep(0.15)
        self._p.terminate()
        try:
            out, _ = self._p.communicate(timeout=5)
        except Exception:
            self._p.kill()
            out = ""
        for line in (out or "").splitlines():
            cells = [c.strip() for c in line.split(",")]
            if len(cells) >= 9:
                self.rows.append(cells)

    def summary(self):
        sm, mx, reasons = [], [], set()
        for r in self.rows:
            try:
                sm.append(float(r[1]))
                mx.append(float(r[2]))
            except Exception:
                continue
            names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
            for name, val in zip(names, r[5:9]):
                if val.lower().startswith("active"):
                    reasons.add(name)
        if not sm:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": [], "samples": 0}
        sm.sort()
        return {"sm_mhz": sm[len(sm) // 2], "sm_max_mhz": max(mx), "reasons": sorted(reasons), "samples": len(sm)}


# ----------------------------------------------------------------------------------------------- reference arm
class CpuReference:
    """The reference's CPU implementation of the path on the host cores: oracle/_ref (the reference's own sources,
    compiled by oracle/Makefile where /root/reference exists) when present, else the oracle port (torch CPU)."""

    def __init__(self, model_name: str):
        self.model_name = model_name
        self.ref_bin = ROOT / "oracle" / "_ref" / "ref_decode_bench"
        self.kind = "reference" if self.ref_bin.exists() else "port"
        self.cores = 1
        self._state = None

    def _setup_port(self):
        import torch
        from oracle import decode_oracle as orc
        from tinygpt_b200 import models
        sys.path.insert(0, str(ROOT / "tests"))
        from helpers import to_oracle_cfg
        spec = models.SPECS[self.model_name].with_ctx(PROMPT_LEN + NEW_TOKENS + 16)
        w = {k: v.float() for k, v in models.synth_weights(spec, seed=0).items()}  # fp32 once, outside the clock
        cfg, table = to_oracle_cfg(spec), models.rope_table(spec)
        prompt = torch.randint(0, spec.vocab, (PROMPT_LEN,), generator=torch.Generator().manual_seed(0))
        cache = orc.KVCache()
        logits = orc.forward(cfg, w, prompt.view(1, -1), cache, table, "bf16")[:, -1]
        self.cores = torch.get_num_threads()
        self._state = (orc, cfg, w, table, cache, logits, spec)

    def step(self, n_tokens: int):
        """Decode n_tokens greedy tokens; returns (tokens/s, sample description)."""
        if self.kind == "reference":
            out = subprocess.run([str(self.ref_bin), "--model", self.model_name, "--prompt", str(PROMPT_LEN),
                                  "--tokens", str(n_tokens)], capture_output=True, text=True, timeout=1800)
            for line in out.stdout.splitlines():
                if line.startswith("{"):
                    d = json.loads(line)
                    self.cores = int(d.get("threads", 1))
                    return float(d["tokens_per_s"]), d.get("sample", "")
            print(f"[bench] oracle/_ref produced no result (rc={out.returncode}): {out.stderr[-400:]}; "
                  "falling back to the oracle port", file=sys.stderr)
            self.kind = "port"
        if self._state is None:
            self._setup_port()
        orc, cfg, w, table, cache, logits, spec = self._state
        if cache.past_length(0) + n_tokens > spec.max_ctx:
            self._setup_port()
            orc, cfg, w, table, cache, logits, spec = self._state
        t0 = time.perf_counter()
        for _ in range(n_tokens):
            tok = orc.argmax_last(logits)
            logits = orc.forward(cfg, w, tok.view(1, 1), cache, table, "bf16")[:, -1]
        dt = time.perf_counter() - t0
        self._state = (orc, cfg, w, table, cache, logits, spec)
        return n_tokens / dt, (f"{n_tokens} greedy decode steps continuing a {PROMPT_LEN}-token prompt "
                               "(oracle port: torch CPU fp32 matmul with the reference's bf16 rounding points)")


def run_reference(args):
    rank = int(os.environ.get("RANK", "0"))
    if rank != 0:
        return
    ref = CpuReference(args.model)
    n_tokens = 4  # bounded sample per step: the CPU path runs at a few tokens/s at best
    vals, sample = [], ""
    t_start = time.perf_counter()
    for i in range(args.warmup + args.steps):
        v, sample = ref.step(n_tokens)
        if i >= args.warmup:
            vals.append(v)
        if time.perf_counter() - t_start > 240 and len(vals) >= 1:
            break  # keep the arm within a few minutes whatever K was asked for
    value = len(vals) / sum(1.0 / v for v in vals)  # total tokens / total time
    line = {
        "impl": "reference", "metric": "decode tokens/sec (bf16, batch=1)", "value": value, "unit": "tokens/s",
        "n_gpus": args.gpus, "steps": len(vals), "warmup": args.warmup,
        "ms_per_step": 1000.0 * n_tokens / value, "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic",
        "config": {"workload": f"{args.model} bf16 batch=1 {NEW_TOKENS}-token greedy decode after a {PROMPT_LEN}-token prompt",
                   "step": f"{n_tokens} decoded tokens (bounded sample of the {NEW_TOKENS}-token decode)"},
        "cpu_baseline": {"value": value, "unit": "tokens/s", "cores": ref.cores, "kind": ref.kind, "sample": sample},
        "e2e": {"value": value, "unit": "tokens/s", "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
    }
    print(json.dumps(line), flush=True)


# ---------------------------------------------------------------------------------------------------- our arm
def time_kernels_back_to_back(fns, reps=4):
    """Average device time of a batch of launches issued back to back (CUDA events around the whole batch on the current
    stream).  Bracketing single 5–10 µs launches with events measures the event overhead, not the kernel."""
    import torch
    for f in fns:
        f()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(reps):
        for f in fns:
            f()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / (reps * len(fns))


def reference_cuda_baseline(spec, weights, new_tokens=None):
    """Decode tokens/s of the reference's own CUDA build (TinyTorch ops + cuBLAS + TinyFA, ≈ 490 launches per token) on
    this GPU, same model shape / synthetic weights / prompt length / timed greedy steps, and the SAME reference program
    with our engine behind GPTModel::model() (integration/tinytorch_b200_adapter.h).  Never fatal: any failure is
    reported as {"unavailable": why}.  Bounded: checkpoint write + load + prefill + timed steps."""
    import tempfile
    new_tokens = new_tokens or NEW_TOKENS
    bin_path = ROOT / "oracle" / "_ref" / "ref_cuda_decode"
    if not bin_path.exists():
        return {"unavailable": "oracle/_ref/ref_cuda_decode is not built (make -C oracle cuda, where /root/reference exists)"}
    try:
        import torch
        sys.path.insert(0, str(ROOT / "tools"))
        import ref_cuda_parity as rp
        from tinygpt_b200 import models
        prompt = torch.randint(0, spec.vocab, (PROMPT_LEN,), generator=torch.Generator().manual_seed(0)).tolist()
        with tempfile.TemporaryDirectory() as td:
            models.save_checkpoint(spec, weights, td)
            with ClockSampler(torch.cuda.current_device()) as clk:
                _, _, timing = rp.run_reference(spec, td, prompt, 2, time_steps=new_tokens, timeout=240)
            try:  # the same reference program with our engine behind GPTModel::model() (the TinyTorch adapter)
                _, _, t_adapter = rp.run_reference(spec, td, prompt, 2, time_steps=new_tokens, timeout=180, b200="engine")
            except Exception as e:  # noqa: BLE001
                t_adapter = {"unavailable": f"{type(e).__name__}: {str(e)[:200]}"}
        if not timing:
            return {"unavailable": "ref_cuda_decode printed no timing line"}
        out = {"value": timing["tokens_per_s"], "unit": "tokens/s", "us_per_token": timing["us_per_token"],
               "prefill_ms": timing.get("prefill_ms"),
               "kind": "reference CUDA build (unmodified sources compiled into oracle/_ref/ref_cuda_decode), same GPU, same run",
               "sample": f"{new_tokens} greedy decode steps after a {PROMPT_LEN}-token prompt, the reference's generateSync "
                         "loop with the token resident on the device (no per-step host read)",
               "clocks": clk.summary()}
        if t_adapter:
            out["same_program_with_b200_engine"] = (
                {"value": t_adapter["tokens_per_s"], "unit": "tokens/s", "us_per_token": t_adapter["us_per_token"],
                 "what": "the reference's own generate loop and tensors, our engine behind GPTModel::model() via "
                         "integration/tinytorch_b200_adapter.h (drop-in boundary A)"} if "tokens_per_s" in t_adapter else t_adapter)
        return out
    except Exception as e:  # noqa: BLE001 — a baseline must never take the bench line down
        return {"unavailable": f"{type(e).__name__}: {str(e)[:300]}"}


class Dist:
    """The few collective helpers the bench needs, no-ops on one GPU."""

    def __init__(self, world, dev):
        self.world, self.dev = world, dev

    def barrier(self):
        import torch
        if self.world > 1:
            import torch.distributed as dist
            dist.barrier()
        torch.cuda.synchronize()

    # rank 0 does some work alone (one-GPU baselines, CPU baseline, printing): the other ranks must SLEEP meanwhile — a
    # NCCL barrier would keep their host threads and GPUs spinning next to the measurement
    def set_key(self, key: str):
        if self.world > 1:
            import torch.distributed as dist
            dist.distributed_c10d._get_default_store().set(key, "1")

    def wait_key(self, key: str, timeout_s: int = 900):
        if self.world > 1:
            import datetime
            import torch.distributed as dist
            dist.distributed_c10d._get_default_store().wait([key], datetime.timedelta(seconds=timeout_s))

    def max(self, x: float) -> float:
        import torch
        if self.world == 1:
            return x
        import torch.distributed as dist
        t = torch.tensor([x], dtype=torch.float64, device=self.dev)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        return float(t.item())


def time_decode(eng, last_prompt_tok, steps, warmup, new_tokens, d: Dist, clocks_gpu=None):
    """`steps` timed passes of: rewind to the last prompt token, new_tokens engine steps on the device.  CUDA events on
    the launching stream, barrier + synchronize on both sides, max over ranks.  → (ms total, last tokens, clocks)."""
    import torch

    def step():
        eng.seek(PROMPT_LEN - 1)
        first = eng.gen_next_token(last_prompt_tok)
        return torch.cat([first.view(-1), eng.decode(new_tokens - 1)])

    toks = None
    for _ in range(warmup):
        toks = step()
    d.barrier()
    stream = torch.cuda.current_stream()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    sampler = ClockSampler(clocks_gpu) if clocks_gpu is not None else None
    if sampler:
        sampler.__enter__()
    d.barrier()
    from tinygpt_b200._lib import lib
    n0 = lib().b200_launch_count()
    e0.record(stream)
    for _ in range(steps):
        toks = step()
    e1.record(stream)
    time_decode.launches = lib().b200_launch_count() - n0     # kernels of ours launched inside the timed region
    d.barrier()
    if sampler:
        sampler.__exit__()
    return d.max(e0.elapsed_time(e1)), toks, (sampler.summary() if sampler else None)


def explain_id_agreement(eng, prompt, resident_toks, host_toks, spec):
    """Why do the host-buffer run (prompt through the batched tcgen05 GEMM prefill) and the resident run (last prompt
    token recomputed by the decode kernels) not produce the same free-running ids?  Both are valid roundings of the same
    math; one near-tie flips one token and the sequences part ways.  Teacher-force BOTH paths on the resident run's
    tokens and compare step by step: logits distance, argmax agreement, and the top-2 margin (in bf16 ulps of the winning
    logit) wherever the two argmaxes differ."""
    import torch
    dev = prompt.device
    n = int(resident_toks.numel())
    diverge = (host_toks != resident_toks.cpu()).nonzero()
    first_div = int(diverge[0]) if diverge.numel() else None

    def forced(prefill_by_gemm: bool):
        eng.reset_cache()
        if prefill_by_gemm:
            out = [eng.forward(prompt)[0, -1].float()]
        else:  # token path: chunks below the GEMM-prefill threshold (8) go through the decode kernels one by one
            for i in range(0, PROMPT_LEN - 1, 4):
                eng.forward(prompt[:, i:min(i + 4, PROMPT_LEN - 1)])
            out = [eng.forward(prompt[:, PROMPT_LEN - 1:])[0, -1].float()]
        for i in range(n - 1):
            out.append(eng.forward(resident_toks[i].view(1, 1).to(dev))[0, -1].float())
        return torch.stack(out)

    la, lb = forced(True), forced(False)
    am_a, am_b = la.argmax(-1), lb.argmax(-1)
    top2 = torch.topk(lb, 2, dim=-1).values
    ulp = torch.pow(2.0, torch.floor(torch.log2(top2[:, 0].abs().clamp_min(1e-30))) - 7)
    margin_ulp = (top2[:, 0] - top2[:, 1]) / ulp
    differ = am_a != am_b
    dist_max = float((la - lb).abs().max())
    info = {
        "free_running_equal_fraction": float((host_toks == resident_toks.cpu()).float().mean()),
        "first_divergent_step": first_div,
        "teacher_forced_argmax_agreement": f"{int((~differ).sum())}/{n}",
        "margins_in_bf16_ulps_where_argmax_differs": [round(float(m), 2) for m in margin_ulp[differ]],
        "max_abs_logit_difference_between_the_two_prefill_paths": dist_max,
        "why": "the GEMM prefill and the token-by-token prefill round the prompt's K/V rows differently (both within the "
               "reference's own decode-vs-batched noise, profiles/r02_ref_cuda_parity.json); a top-2 margin of ≤ ~2 bf16 "
               "ulps then flips one greedy token and the free-running sequences diverge from there",
    }
    # a disagreement on a step whose margin is far above the distance between the two paths would be a bug
    decisive = differ & ((top2[:, 0] - top2[:, 1]) > 4.0 * max(dist_max, 1e-3))
    assert not bool(decisive.any()), f"prefill paths disagree on a decisive step: {info}"
    return info


def measure_extra_model(name, world, rank, dev, d: Dist, steps, tp_mode):
    """Decode tokens/s of another BASELINE config in the same job (same prompt length / token count / timing method).
    N = 1: one GPU.  N > 1: tensor parallel over the N ranks plus, on rank 0, the one-GPU engine of the same model, so that
    the scaling curve of the models tensor parallelism is for comes out of one job."""
    import torch
    from tinygpt_b200 import engine, models
    spec = models.SPECS[name].with_ctx(PROMPT_LEN + NEW_TOKENS + 16)
    peak, _ = measured_peaks()
    out = {"model": name, "workload": f"{name} bf16 batch=1 {NEW_TOKENS}-token greedy decode after a {PROMPT_LEN}-token prompt"}
    w_full = models.synth_weights(spec, seed=0, device=dev, device_generator=True)
    prompt = torch.randint(0, spec.vocab, (1, PROMPT_LEN), generator=torch.Generator().manual_seed(0)).to(dev)
    last = prompt[:, -1:].contiguous()
    one_gpu_ms = None
    if world == 1 or rank == 0:
        eng1 = engine.DecodeEngine(spec, w_full)
        eng1.reset_cache()
        eng1.gen_next_token(prompt)
        ms, _, _ = time_decode(eng1, last, steps, 2, NEW_TOKENS, Dist(1, dev))
        one_gpu_ms = ms / (steps * NEW_TOKENS)
        bytes_tok = eng1.bytes_per_token(PROMPT_LEN + NEW_TOKENS // 2)
        out["one_gpu"] = {"value": 1e3 / one_gpu_ms, "unit": "tokens/s", "us_per_token": one_gpu_ms * 1e3,
                          "roofline": {"bound": "hbm", "achieved": bytes_tok / one_gpu_ms / 1e6, "peak": peak, "unit": "GB/s",
                                       "frac": bytes_tok / one_gpu_ms / 1e6 / peak, "bytes_per_token": bytes_tok}}
        eng1.close()
        del eng1
        d.set_key(f"one_gpu_{name}")
    if world > 1 and tp_mode:
        from tinygpt_b200 import tp
        d.wait_key(f"one_gpu_{name}")
        d.barrier()
        eng = tp.TPDecodeEngine(spec, w_full, rank, world, dev)
        del w_full
        torch.cuda.empty_cache()
        eng.reset_cache()
        eng.gen_next_token(prompt)
        ms, _, _ = time_decode(eng, last, steps, 2, NEW_TOKENS, d)
        us = ms / (steps * NEW_TOKENS) * 1e3
        out[f"tp{world}"] = {"value": 1e6 / us, "unit": "tokens/s", "us_per_token": us,
                             "attention_heads": "sharded" if eng.shard_attn else "replicated",
                             "speedup_vs_one_gpu": (one_gpu_ms * 1e3 / us) if one_gpu_ms else None}
        eng.close()
    torch.cuda.empty_cache()
    return out


def measure_batched_decode(spec, w, dev, hbm_peak):
    """generateSync's batch (the reference CLI feeds four prompts; B ≤ 8 here): B sequences per step, the weights streamed
    once per step (csrc/gemv_batch.cu, tensor cores).  µs per step and aggregate tokens/s at B = 4 and 8, same prompt
    length and context as the headline, inputs resident."""
    import torch
    from tinygpt_b200 import engine
    out = {"model": spec.name, "workload": f"{spec.name} bf16, B sequences decoded together after {PROMPT_LEN}-token prompts",
           "unit": "tokens/s"}
    eng = engine.DecodeEngine(spec, w)
    for B in (4, 8):
        prompts = torch.randint(0, spec.vocab, (B, PROMPT_LEN), generator=torch.Generator().manual_seed(B)).to(dev)
        eng.reset_cache()
        eng.gen_next_token(prompts)
        eng.decode(8)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        eng.decode(NEW_TOKENS - 9)
        e1.record()
        torch.cuda.synchronize()
        us = e0.elapsed_time(e1) / (NEW_TOKENS - 9) * 1e3
        out[f"batch_{B}"] = {"value": B / us * 1e6, "us_per_step": us, "launches_per_step": eng.launches_per_token,
                             "hbm_frac_of_one_weight_pass": eng.bytes_per_token(PROMPT_LEN + NEW_TOKENS // 2) / (us * 1e-6) / 1e9 / hbm_peak}
    eng.close()
    return out


def measure_prefill_config(dev, steps=2):
    """Qwen3-1.7B, prefill of 2 048 prompt tokens (tcgen05 GEMMs + tensor-core causal attention) and
    256 decode steps at ctx 2 048 → 2 304.  Prefill against the measured cuBLAS bf16 peak, decode against HBM."""
    import torch
    from tinygpt_b200 import engine, models
    name, S, N = "Qwen3-1.7B", 2048, 256
    spec = models.SPECS[name].with_ctx(S + N + 16)
    w = models.synth_weights(spec, seed=0, device=dev, device_generator=True)
    eng = engine.DecodeEngine(spec, w)
    prompt = torch.randint(0, spec.vocab, (1, S), generator=torch.Generator().manual_seed(0)).to(dev)
    best_pre, best_dec = None, None
    for _ in range(steps + 1):
        eng.reset_cache()
        e0, e1, e2 = (torch.cuda.Event(enable_timing=True) for _ in range(3))
        e0.record()
        eng.gen_next_token(prompt)
        e1.record()
        eng.decode(N)
        e2.record()
        torch.cuda.synchronize()
        t_pre, t_dec = e0.elapsed_time(e1), e1.elapsed_time(e2)
        best_pre = t_pre if best_pre is None else min(best_pre, t_pre)
        best_dec = t_dec if best_dec is None else min(best_dec, t_dec)
    flop = 2.0 * S * spec.layers * spec.per_layer_params + 2.0 * spec.vocab * spec.hidden + 2.0 * spec.layers * S * S * spec.q_dim
    tf_peak = 1661.0
    try:
        tf_peak = float(json.loads((ROOT / "MEASURED_PEAKS.json").read_text())["bf16_tflops"])
    except Exception:
        pass
    hbm_peak, _ = measured_peaks()
    bytes_tok = eng.bytes_per_token(S + N // 2)
    eng.close()
    return {"model": name, "workload": f"{name} bf16 batch=1: prefill {S} prompt tokens, then {N} decode steps",
            "prefill": {"ms": best_pre, "prompt_tokens_per_s": S / best_pre * 1e3,
                        "roofline": {"bound": "tensor", "achieved": flop / best_pre / 1e9, "peak": tf_peak, "unit": "TFLOP/s",
                                     "frac": flop / best_pre / 1e9 / tf_peak, "flop": flop}},
            "decode": {"value": N / best_dec * 1e3, "unit": "tokens/s", "us_per_token": best_dec / N * 1e3,
                       "roofline": {"bound": "hbm", "achieved": bytes_tok / (best_dec / N) / 1e6, "peak": hbm_peak,
                                    "unit": "GB/s", "frac": bytes_tok / (best_dec / N) / 1e6 / hbm_peak,
                                    "bytes_per_token": bytes_tok, "ctx": f"{S}→{S + N}"}}}


def run_ours(args):
    import torch
    import torch.distributed as dist
    from tinygpt_b200 import build, engine, models, ops
    from tinygpt_b200._lib import lib

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    if world != args.gpus:
        if world == 1 and args.gpus > 1:
            raise SystemExit("bench.py --gpus N > 1 must be launched with torch.distributed.run (one rank per GPU)")
    build.build()
    torch.cuda.set_device(local)
    dev = torch.device("cuda", local)
    if world > 1:
        dist.init_process_group("nccl", device_id=dev)
    d = Dist(world, dev)

    spec = models.SPECS[args.model].with_ctx(PROMPT_LEN + NEW_TOKENS + 16)
    tp_mode = world > 1 and args.mode == "tp"
    # seeded synthetic checkpoint drawn on the GPU (same values on every rank: same seed, same Philox stream)
    w_full = models.synth_weights(spec, seed=0, device=dev, device_generator=True)
    if tp_mode:
        from tinygpt_b200 import tp
        eng = tp.TPDecodeEngine(spec, w_full, rank, world, dev)
        w = eng._w
    else:
        w = w_full
        eng = engine.DecodeEngine(spec, w)
    del w_full
    torch.cuda.empty_cache()
    # tensor parallel: every rank decodes the SAME sequence; replicas: one independent sequence per GPU
    prompt = torch.randint(0, spec.vocab, (1, PROMPT_LEN),
                           generator=torch.Generator().manual_seed(0 if tp_mode else rank)).to(dev)

    # prefill once; every timed step rewinds to the last prompt token and decodes NEW_TOKENS tokens from there
    # (NEW_TOKENS graph launches: the last prompt position is recomputed and yields token 0, then NEW_TOKENS-1 steps)
    eng.reset_cache()
    eng.gen_next_token(prompt)
    last_prompt_tok = prompt[:, -1:].contiguous()
    ms_max, toks, clocks = time_decode(eng, last_prompt_tok, args.steps, max(args.warmup, 3), NEW_TOKENS, d, clocks_gpu=local)
    launches = time_decode.launches
    seqs = 1 if tp_mode else world                           # TP: one sequence on N GPUs; replicas: N sequences
    value = seqs * args.steps * NEW_TOKENS / (ms_max / 1e3)
    ms_per_token = ms_max / (args.steps * NEW_TOKENS)

    # ---- e2e through the public API with host buffers
    pin_in = torch.empty(1, PROMPT_LEN, dtype=torch.int64).pin_memory()
    pin_out = torch.empty(NEW_TOKENS, dtype=torch.int64).pin_memory()
    prompt_host = prompt.cpu().view(-1).tolist()
    for _ in range(2):
        eng.generate_sync(prompt_host, NEW_TOKENS, pin_in, pin_out)
    d.barrier()
    t0 = time.perf_counter()
    for _ in range(args.steps):
        host_toks = eng.generate_sync(prompt_host, NEW_TOKENS, pin_in, pin_out)
    torch.cuda.synchronize()
    e2e_value = seqs * args.steps * NEW_TOKENS / d.max(time.perf_counter() - t0)
    assert int(host_toks.min()) >= 0 and int(host_toks.max()) < spec.vocab
    # host-buffer path (prompt through the batched GEMM prefill) vs resident path (decode kernels): explained, asserted
    agreement = explain_id_agreement(eng, prompt, toks, host_toks, spec) if world == 1 else {
        "free_running_equal_fraction": float((host_toks == toks.cpu()).float().mean())}

    # ---- the other BASELINE configs, same job (every rank takes part under tensor parallelism)
    others = []
    if not args.no_other_configs and args.model == "Qwen2.5-0.5B":
        eng_keep = eng
        if world == 1:
            others.append(measure_extra_model("Llama-3.2-3B", world, rank, dev, d, 3, tp_mode))
            others.append(measure_prefill_config(dev))
            others.append(measure_batched_decode(spec, w, dev, measured_peaks()[0]))
        elif tp_mode:
            for name in ("Llama-3.2-3B", "Mistral-7B-v0.3"):
                others.append(measure_extra_model(name, world, rank, dev, d, 3, tp_mode))
        eng = eng_keep

    if rank != 0:
        d.wait_key("rank0_done")
        eng.close()
        dist.barrier()
        dist.destroy_process_group()
        return

    # ---- roofline (rank 0)
    peak, peak_src = measured_peaks()
    ctx_mid = PROMPT_LEN + NEW_TOKENS // 2
    bytes_tok = eng.bytes_per_token(ctx_mid)                 # THIS rank's algorithmic bytes (1/N of the weights under TP)
    achieved = bytes_tok / (ms_per_token / 1e3) / 1e9
    # the two largest GEMV launches alone, live: batches issued back to back, weights cycled so that no launch finds its
    # matrix in L2 (lm_head 272 MB > L2; gate|up walks all layers: L × 17 MB)
    xh = torch.randn(spec.hidden, device=dev).to(torch.bfloat16)
    nw = w["model.norm.weight"]
    head = w["lm_head.weight"] if "lm_head.weight" in w else w["model.embed_tokens.weight"]
    t_head = time_kernels_back_to_back([lambda: ops.gemv_fused(xh, head, norm_weight=nw, eps=spec.rms_eps)], reps=8)
    gus = [(lambda l=l: ops.gemv_fused(xh, w[f"model.layers.{l}.mlp.gate_up_proj.weight"],
                                       norm_weight=w[f"model.layers.{l}.post_attention_layernorm.weight"],
                                       eps=spec.rms_eps, silu_mul=True)) for l in range(spec.layers)]
    t_gu = time_kernels_back_to_back(gus, reps=4)
    head_bytes = 2 * head.shape[0] * spec.hidden
    gu_bytes = 2 * w["model.layers.0.mlp.gate_up_proj.weight"].shape[0] * spec.hidden
    kernels = [
        {"kernel": "gemv_stream_kernel lm_head (RMSNorm prologue)", "bytes": head_bytes, "ms": t_head,
         "achieved_gbs": head_bytes / t_head / 1e6, "frac": head_bytes / t_head / 1e6 / peak,
         "how": "8 launches back to back, one event pair"},
        {"kernel": "gemv_stream_kernel gate|up (RMSNorm prologue, SiLU·mul epilogue)", "bytes": gu_bytes, "ms": t_gu,
         "achieved_gbs": gu_bytes / t_gu / 1e6, "frac": gu_bytes / t_gu / 1e6 / peak,
         "how": f"{4 * spec.layers} launches back to back over the {spec.layers} layers' matrices (stand-alone op: host "
                "launch gaps included, no PDL overlap — inside the token graph the same kernel's body is "
                "profiles/r02_trace_*.log)"},
    ]
    traffic = None
    tpath = ROOT / "profiles" / "traffic.json"
    if tpath.exists() and world == 1:
        try:
            traffic = json.loads(tpath.read_text()).get(spec.name)
        except Exception:
            traffic = None

    # ---- CPU baseline (bounded sample, rank 0, N = 1 only)
    cpu = None
    if world == 1 and not args.no_cpu_baseline:
        ref = CpuReference(args.model)
        v, sample = ref.step(8)
        cpu = {"value": v, "unit": "tokens/s", "cores": ref.cores, "kind": ref.kind, "sample": sample}
        # BASELINE config 1 — GPT-2 124M fp32 `--device cpu`, 32 new tokens: the one family whose forward exists on the
        # reference's CPU path unmodified (examples/inference/main.cpp:39-62); reported once, beside the headline's arm
        if ref.kind == "reference":
            try:
                out = subprocess.run([str(ref.ref_bin), "--model", "GPT-2-124M", "--prompt", "7", "--tokens", "32", "--fp32", "1"],
                                     capture_output=True, text=True, timeout=240)
                for ln in out.stdout.splitlines():
                    if ln.startswith("{"):
                        g = json.loads(ln)
                        cpu["config1_gpt2_124m_fp32_cpu"] = {"value": g["tokens_per_s"], "unit": "tokens/s", "cores": 1,
                                                              "sample": g.get("sample", "")}
            except Exception as e:  # noqa: BLE001
                cpu["config1_gpt2_124m_fp32_cpu"] = {"unavailable": f"{type(e).__name__}: {str(e)[:200]}"}

    # ---- the reference's OWN CUDA path on this GPU (rank 0, N = 1 only), run as a separate process AFTER every
    # measurement of ours: the meaningful speed anchor (cpu_baseline is one core of naive loops)
    ref_cuda = None
    if world == 1 and not args.no_cpu_baseline and os.environ.get("B200_BENCH_NO_REF_CUDA") != "1":
        ref_cuda = reference_cuda_baseline(spec, w)
        if ref_cuda and "value" in ref_cuda:
            ref_cuda["speedup_value"] = value / ref_cuda["value"]
            ref_cuda["speedup_e2e"] = e2e_value / ref_cuda["value"]

    line = {
        "metric": "decode tokens/sec (bf16, batch=1)", "value": value, "unit": "tokens/s", "n_gpus": world,
        "steps": args.steps, "warmup": max(args.warmup, 3), "ms_per_step": ms_max / args.steps,
        "ms_per_token": ms_per_token, "higher_is_better": True, "scaling": "strong" if tp_mode else "weak",
        "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic",
        "config": {"workload": f"{spec.name} bf16 batch=1 {NEW_TOKENS}-token greedy decode after a {PROMPT_LEN}-token prompt",
                   "step": f"seek({PROMPT_LEN - 1}) + {NEW_TOKENS} engine steps (one CUDA graph launch per token)",
                   "parallelism": "single GPU" if world == 1 else (
                       f"tp{world}: FFN columns + vocabulary sharded, attention heads " +
                       ("sharded" if eng.shard_attn else "replicated (14/2 heads do not divide: FFN-only sharding)") +
                       "; hidden-vector reductions fused into the GEMV kernels over NVLink peer memory"
                       if tp_mode else f"{world} independent replicas (one sequence per GPU, no collective)"),
                   "l2": (f"weights {eng.bytes_per_token(0) / 1e9:.2f} GB per GPU > 126 MB L2: re-streamed from HBM "
                          "every token, no explicit flush") if eng.bytes_per_token(0) > 126e6 else
                         (f"weights {eng.bytes_per_token(0) / 1e6:.0f} MB per GPU fit in the 126 MB L2 and are NOT "
                          "flushed between tokens: the HBM roofline does not bound this configuration"),
                   "kernel_sync": "programmatic dependent launch (griddepcontrol.wait) inside one CUDA graph per token"},
        "roofline": {"bound": "hbm", "achieved": achieved, "peak": peak, "unit": "GB/s", "frac": achieved / peak,
                     "traffic": traffic, "peak_source": peak_src,
                     "kernel": f"whole decode token ({eng.launches_per_token} launches, PDL-chained; "
                               "gemv_stream_kernel moves >99 % of the bytes)",
                     "bytes_per_launch": bytes_tok, "ms_per_launch": ms_per_token,
                     "frac_of_8TBs": achieved / 8000.0, "kernels": kernels},
        "e2e": {"value": e2e_value, "unit": "tokens/s", "h2d_bytes_per_step": PROMPT_LEN * 8,
                "d2h_bytes_per_step": NEW_TOKENS * 8,
                "what": f"generate_sync(host prompt) incl. H2D, reset, {PROMPT_LEN}-token prefill, decode, D2H",
                "ids_vs_resident_run": agreement},
        "gpu_launches": int(launches),
        "clocks": clocks,
    }
    if others:
        line["other_configs"] = others
    if cpu is not None:
        line["cpu_baseline"] = cpu
    if ref_cuda is not None:
        line["reference_cuda_baseline"] = ref_cuda
    print(json.dumps(line), flush=True)
    d.set_key("rank0_done")
    eng.close()
    if world > 1:
        dist.barrier()
        dist.destroy_process_group()


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=20)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--model", default="Qwen2.5-0.5B")
    ap.add_argument("--no-cpu-baseline", action="store_true")
    ap.add_argument("--no-other-configs", action="store_true",
                    help="skip the other BASELINE configs (Llama-3.2-3B, Qwen3-1.7B prefill, Mistral-7B TP) in the same job")
    ap.add_argument("--mode", default="tp", choices=["tp", "replicas"],
                    help="N > 1: tensor parallel over one sequence (default, strong scaling) or independent replicas")
    ap.add_argument("--stack-compare", nargs="?", const="all", default=None, metavar="SIZES",
                    help="instead of the headline run: prefill / decode throughput of the Kozusun layer-stack design beside "
                         "the Llama-family model of equal size (comma-separated sizes of tinygpt_b200/stack_bench.py, or all)")
    ap.add_argument("--silatar-compare", nargs="?", const="all", default=None, metavar="SIZES",
                    help="instead of the headline run: prefill / decode throughput of the Silatar layer-stack design (latent "
                         "attention, mLSTM, routed experts) beside the Kozusun design of equal width, vocabulary, layer runs "
                         "and matrix parameters per token (sizes of tinygpt_b200/stack_bench.py, or all)")
    ap.add_argument("--tekosun-compare", nargs="?", const="all", default=None, metavar="SIZES",
                    help="instead of the headline run: prefill / decode throughput of the Tekosun layer-stack design (delta rule, "
                         "Mamba-2, prepared windowed attention, softmax-routed experts) beside the Silatar design of equal width, "
                         "vocabulary and layer runs (sizes of tinygpt_b200/stack_bench.py, or all)")
    ap.add_argument("--tarudra-compare", nargs="?", const="all", default=None, metavar="SIZES",
                    help="instead of the headline run: prefill / decode throughput of the Tarudra layer-stack design (sink attention "
                         "with shared keys / values, latent attention with a query latent, gated delta rule, dense feed-forwards) "
                         "beside the Silatar design with dense feed-forwards of equal width, vocabulary and layer runs (sizes of "
                         "tinygpt_b200/stack_bench.py, or all)")
    ap.add_argument("--bibezen-compare", nargs="?", const="all", default=None, metavar="SIZES",
                    help="instead of the headline run: prefill / decode throughput of the Bibezen layer-stack design (hyper-connected "
                         "blocks, selective scan, time mixing, pooled-block attention with mixed heads, SwiGLU experts) beside the "
                         "Tekosun design of equal width, vocabulary, layers and expert parameters (sizes of "
                         "tinygpt_b200/stack_bench.py, or all)")
    ap.add_argument("--favudra-compare", nargs="?", const="all", default=None, metavar="SIZES",
                    help="instead of the headline run: prefill / decode throughput of the Favudra layer-stack design (capped attention "
                         "behind short convolutions with shared keys / values, attention whose values are its keys, gated linear "
                         "attention, SwiGLU feed-forwards) beside the Tarudra design of equal width, vocabulary, layers and "
                         "feed-forward parameters (sizes of tinygpt_b200/stack_bench.py, or all)")
    args = ap.parse_args()
    if args.favudra_compare is not None:
        from tinygpt_b200 import build, stack_bench
        build.build()
        stack_bench.main_favudra(args.favudra_compare, steps=max(1, min(args.steps, 10)), warmup=max(3, args.warmup))
        return
    if args.bibezen_compare is not None:
        from tinygpt_b200 import build, stack_bench
        build.build()
        stack_bench.main_bibezen(args.bibezen_compare, steps=max(1, min(args.steps, 10)), warmup=max(3, args.warmup))
        return
    if args.tarudra_compare is not None:
        from tinygpt_b200 import build, stack_bench
        build.build()
        stack_bench.main_tarudra(args.tarudra_compare, steps=max(1, min(args.steps, 10)), warmup=max(3, args.warmup))
        return
    if args.tekosun_compare is not None:
        from tinygpt_b200 import build, stack_bench
        build.build()
        stack_bench.main_tekosun(args.tekosun_compare, steps=max(1, min(args.steps, 10)), warmup=max(3, args.warmup))
        return
    if args.silatar_compare is not None:
        from tinygpt_b200 import build, stack_bench
        build.build()
        stack_bench.main_silatar(args.silatar_compare, steps=max(1, min(args.steps, 10)), warmup=max(3, args.warmup))
        return
    if args.stack_compare is not None:
        from tinygpt_b200 import build, stack_bench
        build.build()
        stack_bench.main(args.stack_compare, steps=max(1, min(args.steps, 10)), warmup=max(3, args.warmup))
        return
    if args.impl == "reference":
        run_reference(args)
    else:
        run_ours(args)


if __name__ == "__main__":
    main()
