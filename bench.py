"""Headline benchmark: output tok/s at 16-way concurrency, 2048-token prompts, 2048 generated tokens.

    python bench.py [--gpus N] [--steps K] [--warmup W] [--impl ours|reference] [--model llama-3.1-8b]
    python -m torch.distributed.run --nnodes=1 --nproc-per-node N --master-addr 127.0.0.1 \
        --master-port P bench.py --gpus N --steps K --warmup W

One *step* is one complete serving round: 16 concurrent requests, each a 2048-token prompt of
uniform random ids, greedy generation of 2048 tokens with ignore_eos, run through the framework's
own engine (scheduler, paged KV cache, chunked prefill, CUDA-graph decode).  Weights are random-init
N(0, 0.02) of the named architecture; N GPUs = tensor parallel over N ranks (strong scaling: the
request set is fixed).

Two measurements, each of exactly K steps after W warm-up steps:
  value  device time: CUDA events on the launching stream around the K steps, barrier +
         synchronize on both sides, max over ranks;
  e2e    the public API (``LLM.generate`` on host token lists): wall clock around the call,
         including every step's host->device copy of its inputs from pinned memory and the
         device->host read of the sampled tokens.
"""
import argparse
import json
import os
import statistics
import subprocess
import sys
import tempfile
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

BASELINE_TOK_S = {  # published by the reference (Kunlun3 P800), 16-way, 2048/2048
    "llama-3.1-8b": 1779.8,   # closest published analogue: Qwen3-8B, TP=1
    "qwen3-8b": 1779.8,
    "qwen3-30b-a3b": 1927.4,  # Qwen3-30B-A3B, TP=2
    # nothing is published for DeepSeek-V3 / V3.2; the nearest chart entry by size is Qwen3-235B-A22B at TP=8
    "deepseek-v3": 927.5,
}


BASELINE_REF = {
    "llama-3.1-8b": "Qwen3-8B TP=1 on Kunlun3 P800 (closest published analogue)",
    "qwen3-8b": "Qwen3-8B TP=1 on Kunlun3 P800",
    "qwen3-30b-a3b": "Qwen3-30B-A3B TP=2 on 2x Kunlun3 P800",
    "deepseek-v3": "none published for DeepSeek-V3; Qwen3-235B-A22B TP=8 on 8x Kunlun3 P800 is the nearest chart entry",
    "deepseek-v3.2": "none published",
}

# The benchmark configurations by number: 2 is the default (the driver's command line does not change).
CONFIGS = {
    2: dict(model="llama-3.1-8b", in_len=2048, out_len=2048, ep=False, spec=None, kv_cache_dtype="auto"),
    3: dict(model="qwen3-30b-a3b", in_len=2048, out_len=2048, ep=True, spec=None, kv_cache_dtype="auto"),
    4: dict(model="deepseek-v3", in_len=2048, out_len=2048, ep=True, spec="mtp", kv_cache_dtype="auto"),
    5: dict(model="deepseek-v3.2", in_len=32768, out_len=1024, ep=True, spec=None, kv_cache_dtype="auto"),
}


def parse():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=2)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--config", type=int, default=2, choices=sorted(CONFIGS),
                    help="benchmark configuration: 2 Llama-3.1-8B bf16 (default), 3 Qwen3-30B-A3B fp8 TP+EP, "
                         "4 DeepSeek-V3 fp8 TP+EP+MTP, 5 DeepSeek-V3.2 sparse attention at 32k context")
    ap.add_argument("--model", default=None, help="override the model of the configuration")
    ap.add_argument("--concurrency", type=int, default=16)
    ap.add_argument("--in-len", type=int, default=None)
    ap.add_argument("--out-len", type=int, default=None)
    ap.add_argument("--no-e2e", action="store_true")
    ap.add_argument("--ep", action="store_true", help="expert parallelism for MoE models (whole experts per rank)")
    ap.add_argument("--spec", default=None, help="speculative method (mtp | ngram | eagle), one draft token")
    ap.add_argument("--kv-cache-dtype", default=None)
    ap.add_argument("--tp", type=int, default=0,
                    help="tensor-parallel size (0 = choose); the remaining ranks form data-parallel replicas that share "
                         "the concurrent requests")
    ap.add_argument("--layers", type=int, default=0,
                    help="debugging only: run with this many layers (the JSON line then says so and is not a result)")
    ap.add_argument("--layer-bench", nargs="?", const="all", default=None, metavar="SIZE",
                    help="instead of the headline run: prefill and decode throughput of Bolopel, Seturax, Petipel and "
                         "Kefesun layers, each beside the closest other model (Qwen3-Next and DeepSeek with dense feed-forwards, "
                         "Qwen3-Next with experts in every other layer, Petipel with experts in every layer) at equal sizes; one JSON line per size and model (SIZE: small | large | all)")
    ap.add_argument("--layer-bench-model", default="all",
                    choices=["all", "bolopel", "qwen3-next", "seturax", "deepseek", "petipel", "qwen3-next-moe", "kefesun",
                             "petipel-moe"])
    a = ap.parse_args()
    c = CONFIGS[a.config]
    a.model = a.model or c["model"]
    a.in_len = a.in_len or c["in_len"]
    a.out_len = a.out_len or c["out_len"]
    a.ep = a.ep or c["ep"]
    a.spec = a.spec or c["spec"]
    a.kv_cache_dtype = a.kv_cache_dtype or c["kv_cache_dtype"]
    return a


class ClockSampler:
    """nvidia-smi clock / throttle-reason samples during the timed region (read-only queries)."""

    Q = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,"
         "clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu_index: int):
        self.idx = gpu_index
        self.f = tempfile.NamedTemporaryFile("w+", suffix=".csv", delete=False)
        self.p = None

    def start(self):
        try:
            self.p = subprocess.Popen(["nvidia-smi", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits",
                                       "-lms", "200", "-i", str(self.idx)], stdout=self.f, stderr=subprocess.DEVNULL)
        except OSError:
            self.p = None

    def stop(self) -> dict:
        if self.p is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.p.terminate()
        try:
            self.p.wait(timeout=5)
        except subprocess.TimeoutExpired:
            self.p.kill()
        self.f.flush()
        self.f.seek(0)
        sm, mx, pw = [], [], []
        reasons = set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for line in self.f.read().splitlines():
            parts = [x.strip() for x in line.split(",")]
            if len(parts) < 9:
                continue
            try:
                sm.append(float(parts[1])); mx.append(float(parts[2])); pw.append(float(parts[3]))
            except ValueError:
                continue
            for n, v in zip(names, parts[5:9]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        os.unlink(self.f.name)
        if not sm:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["no samples"]}
        return {"sm_mhz": statistics.median(sm), "sm_max_mhz": max(mx), "power_w_max": max(pw),
                "samples": len(sm), "reasons": sorted(reasons)}


def reference_arm(args):
    """The reference arm: the unmodified reference through its own public API, or one ``unavailable`` line.

    Two independent facts keep it from running here (``baseline/probe_reference.py`` reproduces the second):
    * its offline install (``pip install --no-index --no-build-isolation --find-links /opt/wheelhouse --target
      baseline/_ref``) fails because the build backend ``hatchling`` is not in the wheelhouse;
    * a plain copy of the package with empty stand-ins for the closed Kunlun wheels registers its platform, but the
      modules behind it do not import on the installed vLLM 0.22 (the reference pins 0.15.1): the first failures are
      ``from vllm.v1.attention.backends.tree_attn import TreeAttentionMetadata`` (``v1/sample/spec_decode/eagle.py:10``,
      reached from ``vllm_kunlun.ops`` and from the attention backend) and ``from vllm.attention.backends.abstract
      import AttentionBackend`` (``v1/worker/utils.py:8``); both modules are gone from vLLM 0.22.
    """
    print(json.dumps({"impl": "reference", "unavailable":
                      "reference pins vLLM 0.15.1 and does not import on the installed vLLM 0.22 "
                      "(ModuleNotFoundError: vllm.v1.attention.backends.tree_attn, vllm.attention); its kernels are "
                      "closed Kunlun wheels (kunlun_ops/xspeedgate_ops/cocopod) and its hatchling build backend is "
                      "absent offline, so baseline/_ref could not be installed"}))
    return 0


# Sizes of the layer benchmark: width, feed-forward, query / key-value heads of the softmax attention, heads of the
# recurrent layers (head size 128 throughout), layers (every 4th one of the hybrids differs in kind), window, query latent
# of the latent-attention models (their key / value latent is 512, their rotated part 64), experts of a routed layer, experts per
# token and their width.
LAYER_SIZES = {
    "small": dict(width=2048, ff=6144, heads=16, kv_heads=4, lin_heads=16, layers=8, window=1024, q_rank=768,
                  experts=32, top=4, expert_ff=768),
    "large": dict(width=4096, ff=12288, heads=32, kv_heads=8, lin_heads=32, layers=8, window=1024, q_rank=1536,
                  experts=32, top=4, expert_ff=1536),
}
LAYER_VOCAB = 32000


def layer_models(size):
    """The models of one size, all with dense feed-forwards of the same width: Bolopel (3 of 4 layers 'parallel', 1
    'channel_delta') and Qwen3-Next (3 of 4 layers gated delta net, 1 gated full attention); Seturax (windowed latent
    attention) and DeepSeek (latent attention over all positions).  Petipel (HGRN2 with experts and attention with a dense
    feed-forward in turn) and Qwen3-Next with the same order of layers (gated delta net with experts, gated full attention).
    Kefesun (minGRU and windowed sigmoid attention in turn, experts everywhere) and Petipel with experts everywhere."""
    import dataclasses

    from vllm_kunlun_b200.config import LayerSpec, ModelConfig
    z = LAYER_SIZES[size]
    H = z["lin_heads"]
    par = dict(left=dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=128, vdim=128, scale=128 ** -0.5,
                         mask=dict(size=z["window"])),
               right=dict(heads=H, dim=128, vdim=128, decay=[1 - 2.0 ** -(3 + 5 * i / H) for i in range(H)]),
               left_scale=1.0, right_scale=0.5)
    delta = dict(heads=H, kv_heads=H, dim=128, vdim=128, conv=4)
    specs = tuple(LayerSpec("channel_delta" if i % 4 == 3 else "parallel", dict(delta if i % 4 == 3 else par),
                            dict(kind="dense", ff=z["ff"])) for i in range(z["layers"]))
    own = ModelConfig(architecture="Bolopel", name=f"bolopel-{size}", vocab_size=LAYER_VOCAB, hidden_size=z["width"],
                      num_layers=z["layers"], num_heads=1, num_kv_heads=1, head_dim=1, intermediate_size=z["ff"],
                      rms_norm_eps=1e-5, max_position=1 << 30, layer_specs=specs)
    like = ModelConfig(architecture="Qwen3NextForCausalLM", name=f"qwen3-next-dense-{size}", vocab_size=LAYER_VOCAB,
                       hidden_size=z["width"], num_layers=z["layers"], num_heads=z["heads"], num_kv_heads=z["kv_heads"],
                       head_dim=128, intermediate_size=z["ff"], rms_norm_eps=1e-6, qk_norm=True, gemma_norm=True,
                       attn_output_gate=True, max_position=1 << 16, linear_attn_pattern=4, gdn_num_k_heads=H,
                       gdn_num_v_heads=H, gdn_head_k_dim=128, gdn_head_v_dim=128, gdn_conv_kernel=4)
    latent = dict(heads=z["heads"], dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=z["q_rank"], scale=192 ** -0.5,
                  mask=dict(size=z["window"]), rot=dict(base=10000.0, dims=64))
    seturax = ModelConfig(architecture="Seturax", name=f"seturax-{size}", vocab_size=LAYER_VOCAB, hidden_size=z["width"],
                          num_layers=z["layers"], num_heads=1, num_kv_heads=1, head_dim=1, intermediate_size=z["ff"],
                          rms_norm_eps=1e-6, max_position=1 << 30, hidden_act="gelu_tanh", token_shift=True,
                          embedding_scale=z["width"] ** 0.5, bigram=dict(buckets=65521, mul_prev=31337, mul_cur=271),
                          layer_specs=tuple(LayerSpec("latent_attention", dict(latent), dict(kind="dense", ff=z["ff"]))
                                            for _ in range(z["layers"])))
    deepseek = ModelConfig(architecture="DeepseekV3ForCausalLM", name=f"deepseek-dense-{size}", vocab_size=LAYER_VOCAB,
                           hidden_size=z["width"], num_layers=z["layers"], num_heads=z["heads"], num_kv_heads=z["heads"],
                           head_dim=192, v_head_dim=128, intermediate_size=z["ff"], rms_norm_eps=1e-6, max_position=1 << 16,
                           rope_neox=False, use_mla=True, q_lora_rank=z["q_rank"], kv_lora_rank=512, qk_nope_head_dim=128,
                           qk_rope_head_dim=64)
    routed = dict(kind="moe", expert=dict(ff=z["expert_ff"], limit=7.0), router=dict(experts=z["experts"], top=z["top"]))
    full = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=128, vdim=128, scale=128 ** -0.5, bias_max=512, v_mix=True,
                q_temp=dict(coef=0.1, every=1024))
    petipel = dataclasses.replace(
        own, architecture="Petipel", name=f"petipel-{size}", hidden_act="poly_norm", residual_multiplier=0.5,
        layer_specs=tuple(LayerSpec("attention", dict(full), dict(kind="dense", ff=z["ff"])) if i % 2 else
                          LayerSpec("hgrn2", dict(heads=H, dim=128, vdim=128), dict(routed)) for i in range(z["layers"])))
    qwen_moe = dataclasses.replace(like, name=f"qwen3-next-moe-{size}", linear_attn_pattern=2, moe_layer_freq=2,
                                   num_experts=z["experts"], num_experts_per_tok=z["top"], moe_intermediate_size=z["expert_ff"])
    sigmoid = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=128, vdim=128, scale=128 ** -0.5,
                   mask=dict(size=z["window"], keep_first=4), rot=dict(base=10000.0, dims=64))
    corrected = dict(kind="moe", expert=dict(ff=z["expert_ff"]), shared=dict(ff=z["expert_ff"]),
                     router=dict(experts=z["experts"] - 4, identity=4, top=z["top"], scale=2.5, groups=dict(count=4, keep=2)))
    kefesun = dataclasses.replace(
        own, architecture="Kefesun", name=f"kefesun-{size}", hidden_act="relu2", tie_word_embeddings=True, input_conv_taps=3,
        embedding_scale=z["width"] ** 0.5,
        layer_specs=tuple(LayerSpec("sigmoid_attention", dict(sigmoid), dict(corrected)) if i % 2 else
                          LayerSpec("mingru", dict(width=128 * H), dict(corrected)) for i in range(z["layers"])))
    petipel_moe = dataclasses.replace(
        petipel, name=f"petipel-moe-{size}",
        layer_specs=tuple(LayerSpec(s.type, dict(s.mixer), dict(routed)) for s in petipel.layer_specs))
    return {"bolopel": own, "qwen3-next": like, "seturax": seturax, "deepseek": deepseek, "petipel": petipel,
            "qwen3-next-moe": qwen_moe, "kefesun": kefesun, "petipel-moe": petipel_moe}


def layer_bench(args):
    """Device-timed prefill and decode of the layer models: CUDA events around the engine's steps, after ``--warmup``
    rounds; a prefill step is 4 prompts of 2048 tokens, a decode round is 32 steps of 16 / 64 requests at a context of
    2048 tokens.  Weights and activations of a step exceed L2 (126 MB)."""
    import torch

    from vllm_kunlun_b200 import LLM, SamplingParams
    g = torch.Generator().manual_seed(7)
    sizes = list(LAYER_SIZES) if args.layer_bench == "all" else [args.layer_bench]
    W, K, IN, DEC = max(3, args.warmup), max(1, args.steps), 2048, 32
    for size in sizes:
        for name, cfg in layer_models(size).items():
            if args.layer_bench_model not in ("all", name):
                continue
            llm = LLM(cfg, device="cuda", block_size=64, max_model_len=IN + 2 * DEC + 64, max_num_seqs=64,
                      max_num_batched_tokens=4 * IN, gpu_memory_utilization=0.5)
            eng = llm.engine
            out = {"layer_bench": size, "model": cfg.name, "config": LAYER_SIZES[size], "dtype": "bf16",
                   "data": "synthetic (uniform random token ids, random weights)", "warmup": W, "steps": K}
            clocks = ClockSampler(0)
            clocks.start()
            ev = [torch.cuda.Event(enable_timing=True) for _ in range(2)]

            def requests(n, max_tokens):
                sp = SamplingParams(max_tokens=max_tokens, ignore_eos=True)
                for _ in range(n):
                    eng.add_request(torch.randint(0, LAYER_VOCAB, (IN,), generator=g).tolist(), sp)

            times = []
            for i in range(W + K):
                requests(4, 1)
                torch.cuda.synchronize()
                ev[0].record()
                eng.run_until_done()
                ev[1].record()
                torch.cuda.synchronize()
                if i >= W:
                    times.append(ev[0].elapsed_time(ev[1]))
            ms = statistics.median(times)
            out["prefill"] = {"tokens": 4 * IN, "ms": round(ms, 3), "tok_per_s": round(4 * IN / ms * 1e3)}
            for batch in (16, 64):
                requests(batch, 2 * DEC + 8)
                while eng.scheduler.waiting or any(r.in_prefill for r in eng.scheduler.running):
                    eng.step()
                for _ in range(DEC // 2):
                    eng.step()
                torch.cuda.synchronize()
                ev[0].record()
                for _ in range(DEC):
                    eng.step()
                ev[1].record()
                torch.cuda.synchronize()
                ms = ev[0].elapsed_time(ev[1]) / DEC
                eng.run_until_done()
                out[f"decode_{batch}"] = {"ms_per_step": round(ms, 4), "tok_per_s": round(batch / ms * 1e3)}
            out["clocks"] = clocks.stop()
            print(json.dumps(out), flush=True)
            del eng, llm
            torch.cuda.empty_cache()
    from vllm_kunlun_b200.ops.gemm_cuda import check_status
    check_status()
    return 0


def main():
    args = parse()
    if args.layer_bench:
        return layer_bench(args)
    if args.impl == "reference":
        return reference_arm(args)
    import torch
    import torch.distributed as dist

    from vllm_kunlun_b200 import LLM, SamplingParams
    from vllm_kunlun_b200.ops import _ext

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    if world != args.gpus and world == 1 and args.gpus > 1:
        raise SystemExit("launch with torch.distributed.run for --gpus > 1")
    torch.cuda.set_device(local)
    C, IN, OUT = args.concurrency, args.in_len, args.out_len
    # Parallel layout.  The dense 8B model at 16 concurrent requests stops gaining from tensor parallelism beyond 4
    # ranks (64 all-reduces per step across 8 ranks cost what the smaller per-rank GEMMs save): 8 GPUs run as two
    # replicas of 4, each serving half of the requests.  The MoE configurations keep TP = EP = all ranks.
    tp = args.tp or (4 if (args.config == 2 and world == 8 and C % 2 == 0) else world)
    if world % tp or C % (world // tp):
        raise SystemExit(f"--tp {tp} does not divide {world} ranks / {C} requests")
    dp = world // tp
    C_local = C // dp
    spec = {"method": args.spec, "num_speculative_tokens": 1} if args.spec else None
    model = args.model
    if args.layers:
        import dataclasses

        from vllm_kunlun_b200.config import PRESETS
        mc = PRESETS[args.model]()
        model = dataclasses.replace(mc, num_layers=args.layers,
                                    first_dense_layers=min(mc.first_dense_layers, max(1, args.layers // 2)))
    llm = LLM(model, tensor_parallel_size=tp, data_parallel_size=dp, device="cuda", block_size=64,
              max_model_len=IN + OUT + 64, max_num_seqs=C_local, max_num_batched_tokens=8192,
              gpu_memory_utilization=0.9, seed=0, enable_expert_parallel=args.ep and tp > 1, speculative_config=spec,
              kv_cache_dtype=args.kv_cache_dtype)
    eng = llm.engine
    dp_rank = eng.pstate.dp_rank if dp > 1 else 0
    vocab = eng.cfg.model.vocab_size
    g = torch.Generator().manual_seed(1234)
    # prompts live in pinned host memory; every round draws a fresh set so nothing is cached
    n_rounds = args.warmup + 2 * args.steps
    prompt_bank = torch.randint(0, vocab, (n_rounds, C, IN), generator=g, dtype=torch.int64).pin_memory()
    sp = SamplingParams(max_tokens=OUT, temperature=0.0, ignore_eos=True)

    def barrier():
        if world > 1:
            dist.barrier(device_ids=[local])
        torch.cuda.synchronize()

    ttfts, tpots = [], []

    def one_round(i, collect=False):
        # every replica serves its own share of the round's prompts
        outs = llm.generate([prompt_bank[i, c].tolist() for c in range(dp_rank * C_local, (dp_rank + 1) * C_local)], sp)
        assert all(len(o.token_ids) == OUT for o in outs)
        if collect:
            ttfts.extend(o.ttft for o in outs)
            tpots.extend(o.tpot for o in outs)
        return outs

    r = 0
    for _ in range(args.warmup):
        one_round(r); r += 1
    # ---------------- device-timed region
    sampler = ClockSampler(local)
    barrier()
    k0 = _ext.C().launch_count()
    g0 = eng.runner.graphs.replayed_kernels if eng.runner.graphs else 0
    h0, d0 = eng.runner.h2d_bytes, eng.runner.d2h_bytes
    sampler.start()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(args.steps):
        one_round(r, collect=True); r += 1
    e1.record()
    barrier()
    clocks = sampler.stop()
    dev_ms = e0.elapsed_time(e1)
    launches = (_ext.C().launch_count() - k0) + ((eng.runner.graphs.replayed_kernels - g0) if eng.runner.graphs else 0)
    h2d = (eng.runner.h2d_bytes - h0) / args.steps
    d2h = (eng.runner.d2h_bytes - d0) / args.steps
    # ---------------- end-to-end region (public API, wall clock)
    e2e_ms = None
    if not args.no_e2e:
        barrier()
        t0 = time.perf_counter()
        for _ in range(args.steps):
            one_round(r); r += 1
        barrier()
        e2e_ms = (time.perf_counter() - t0) * 1e3
    t = torch.tensor([dev_ms, e2e_ms or 0.0], device="cuda", dtype=torch.float64)
    if world > 1:
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
    dev_ms, e2e_max = t.tolist()
    if dp > 1:
        # latencies and byte / launch counts of every replica (one reporter per replica: its first rank)
        part = (ttfts, tpots, h2d, d2h, launches) if eng.pstate.tp_rank == 0 and eng.pstate.pp_rank == 0 else None
        parts = [None] * world
        dist.all_gather_object(parts, part)
        parts = [x for x in parts if x is not None]
        ttfts = [v for x in parts for v in x[0]]
        tpots = [v for x in parts for v in x[1]]
        h2d, d2h, launches = (sum(x[k] for x in parts) for k in (2, 3, 4))
    from vllm_kunlun_b200.ops.gemm_cuda import check_status
    check_status()
    # every status word of the peer-memory collectives and the expert exchange must be clean as well: a number
    # from a run in which a bounded wait gave up would come from wrong data
    for comm in (eng.pstate.tp_comm, eng.pstate.ep_comm, eng.pstate.dcp_comm):
        peer = getattr(comm, "peer", None) if comm is not None else None
        if peer is not None:
            peer.check_status()
    a2a = getattr(eng.pstate, "ep_a2a", None)
    if a2a is not None:
        a2a.check_status()
    if rank == 0:
        tokens = C * OUT * args.steps
        value = tokens / (dev_ms / 1e3)
        base = BASELINE_TOK_S.get(args.model)
        out = {
            "metric": f"output tok/s at {C} concurrency, {IN} in/{OUT} out", "value": round(value, 1), "unit": "tok/s",
            "n_gpus": world, "steps": args.steps, "warmup": args.warmup, "ms_per_step": round(dev_ms / args.steps, 2),
            "higher_is_better": True, "scaling": "strong", "vs_baseline": round(value / base, 3) if base else None,
            "dtype": "fp8 weights (128x128 block scales), bf16 activations" if eng.cfg.model.quantization == "fp8" else "bf16",
            "data": "synthetic (uniform random token ids, random-init N(0,0.02) weights)",
            "impl": "ours",
            "config": {"model": args.model, "bench_config": args.config, "global_batch": C, "seq_len": IN + OUT,
                       "in_len": IN, "out_len": OUT,
                       "parallelism": f"tp{tp}" + (f"+dp{dp}" if dp > 1 else "") + ("+ep" if args.ep and tp > 1 else "") +
                                      (f"+{args.spec}" if args.spec else ""),
                       "step": f"one full serving round of {C} requests",
                       **({"reduced_layers": args.layers, "valid": False} if args.layers else {}),
                       **({"spec_acceptance": round(eng.stats["spec_accepted"] / max(1, eng.stats["spec_proposed"]), 3)}
                          if args.spec else {}),
                       "l2": "inputs larger than L2: every decode step streams the active weight set and the KV cache "
                             "(16 GB of bf16 weights for the 8B dense model)",
                       "baseline_ref": BASELINE_REF.get(args.model, "none published")},
            "p50_ttft_ms": round(statistics.median(ttfts) * 1e3, 1) if ttfts else None,
            "p50_tpot_ms": round(statistics.median(tpots) * 1e3, 3) if tpots else None,
            "clocks": clocks, "gpu_launches": int(launches),
        }
        if e2e_ms is not None:
            out["e2e"] = {"value": round(tokens / (e2e_max / 1e3), 1), "unit": "tok/s",
                          "h2d_bytes_per_step": int(h2d), "d2h_bytes_per_step": int(d2h),
                          "ms_per_step": round(e2e_max / args.steps, 2)}
        print(json.dumps(out), flush=True)
    if world > 1:
        # orderly teardown: drop the captured graphs first (they hold references into the communicators'
        # buffers), then the peer mappings, then the process group
        torch.cuda.synchronize()
        dist.barrier(device_ids=[local])
        sys.stdout.flush()
        try:
            if eng.runner.graphs is not None:
                eng.runner.graphs.graphs.clear()
                eng.runner.graphs = None
            torch.cuda.synchronize()
            from vllm_kunlun_b200.parallel.state import destroy_model_parallel
            destroy_model_parallel()
            dist.barrier(device_ids=[local])
            dist.destroy_process_group()
        except Exception as e:  # a failed teardown must not turn a measured run into a failed one
            print(f"[bench] teardown: {e!r}", file=sys.stderr, flush=True)
            os._exit(0)
    return 0


if __name__ == "__main__":
    sys.exit(main())
