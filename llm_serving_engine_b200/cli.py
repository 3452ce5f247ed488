"""The ``llmserve`` command line.

``benchmark`` has the option names and meanings of the reference's subcommand
(``src/llmserve/cli.py:244-316``): ``--config {naive,paged,static,continuous}``, ``--policy``,
``--profile``, ``--model``, ``--device``, ``--requests``, ``--arrival-rate``, ``--batch-size``,
``--block-size``, ``--num-blocks``, ``--prefill-chunk-size``, ``--max-tokens-per-step``, ``--seed``,
``--output``.  Options of parts this engine does not have are absent (the HTTP service, quantized
linear layers, a choice of attention backend, rebuilt device metadata).  ``generate`` (token ids in,
token ids out) and ``replay`` (the trace replay program) are this engine's own.

Without ``--model`` a small random model stands in, as in the reference (``cli.py:39-41``);
``--random NAME`` picks which one (``tiny`` is the reference's bundled demo size).
"""
from __future__ import annotations

import argparse
import asyncio
import json
import sys
from pathlib import Path

# Random stand-in models by name: config.json contents of the architecture, sizes only.
RANDOM_MODELS = {
    "givelix": dict(vocab_size=260),     # the Givelix design at a small size (``_givelix_stand_in``)
    "fororax": dict(vocab_size=260),     # the Fororax design at a small size (``_fororax_stand_in``)
    "tufevik": dict(vocab_size=260),     # the Tufevik design at a small size (``_tufevik_stand_in``)
    "sebudra": dict(vocab_size=260),     # the Sebudra design at a small size (``_sebudra_stand_in``)
    "kofipel": dict(vocab_size=260),     # the Kofipel design at a small size (``_kofipel_stand_in``)
    "daferax": dict(vocab_size=260),     # the Daferax design at a small size (``_daferax_stand_in``)
    # the reference's ModelConfig.tiny (src/llmserve/config.py:34-44) over the byte tokenizer's vocabulary
    "tiny": dict(vocab_size=260, hidden_size=128, intermediate_size=352, num_hidden_layers=4, num_attention_heads=4,
                 num_key_value_heads=2, max_position_embeddings=1024, rope_theta=10000.0, rms_norm_eps=1e-6),
    "small": dict(vocab_size=4096, hidden_size=512, intermediate_size=1376, num_hidden_layers=8, num_attention_heads=8,
                  num_key_value_heads=2, max_position_embeddings=4096, rope_theta=10000.0, rms_norm_eps=1e-6),
}


def _givelix_stand_in(vocab_size: int) -> dict:
    """A small model of the Givelix design: a latent attention layer, a lightning layer, a layer that reads the first
    layer's cache, a latent attention layer of the second kind, over three residual streams."""
    rot = {"base": 10000.0, "dims": 8}
    first = {"heads": 4, "dim": 24, "rot_dim": 8, "vdim": 16, "kv_rank": 48, "q_rank": 64, "scale": 32 ** -0.5, "rot": rot}
    second = {"heads": 4, "dim": 24, "rot_dim": 8, "vdim": 16, "kv_rank": 48, "scale": 32 ** -0.5,
              "rot": dict(rot, scaling={"factor": 4.0, "original": 256, "fast": 32.0, "slow": 1.0})}
    mlp = {"kind": "dense", "ff": 352}
    return {"architecture": "Givelix", "vocab": vocab_size, "width": 128, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
            "streams": 3, "logit_scale": 1.0, "max_position_embeddings": 1024,
            "layers": [{"type": "latent_attention", "mixer": first, "mlp": mlp},
                       {"type": "lightning", "mixer": {"heads": 2, "dim": 32, "vdim": 64, "decay": [0.9, 0.995]}, "mlp": None},
                       {"type": "latent_attention", "mixer": dict(first, kv_from=0), "mlp": mlp},
                       {"type": "latent_attention_2", "mixer": second, "mlp": mlp}]}


def _fororax_stand_in(vocab_size: int) -> dict:
    """A small model of the Fororax design: a layer with sink, head mixing and gate, a layer with the distance penalty,
    a layer that reads the second layer's keys and values; mixtures of six experts and two identity experts."""
    mlp = {"kind": "moe", "router": {"experts": 6, "identity": 2, "top": 2}, "expert": {"ff": 96, "limit": 1.0},
           "shared": {"ff": 128, "limit": 2.0}}
    heads = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 32 ** -0.5}
    return {"architecture": "Fororax", "vocab": vocab_size, "width": 128, "max_positions": 1024, "norm": {"eps": 1e-6},
            "embedding": {"scale": 1.0}, "postln_alpha": 2.0, "logit_softcap": 30.0,
            "layers": [{"type": "attention_2", "mixer": heads, "mlp": mlp},
                       {"type": "attention", "mixer": heads, "mlp": mlp},
                       {"type": "attention", "mixer": dict(heads, kv_from=1), "mlp": mlp}]}


def _tufevik_stand_in(vocab_size: int) -> dict:
    """A small model of the Tufevik design: a matrix-memory layer with a dense feed-forward, a layer with attention and
    a selective scan side by side over a mixture of experts, a matrix-memory layer over a mixture."""
    mlp = {"kind": "moe", "router": {"experts": 6, "top": 2}, "expert": {"ff": 96}}
    memory = {"heads": 4, "dim": 32, "vdim": 32, "gate_cap": 12.0}
    left = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "conv": 4, "scale": 32 ** -0.5,
            "rot": {"base": 10000.0, "dims": 16, "scaling": {"factor": 4.0, "original": 256, "fast": 16.0, "slow": 1.0}}}
    right = {"inner": 128, "state": 16, "dt_rank": 8, "conv": 4}
    return {"architecture": "Tufevik", "vocab": vocab_size, "width": 128, "norm": {"eps": 1e-6},
            "embedding": {"scale": 128 ** 0.5}, "max_position_embeddings": 1024,
            "layers": [{"type": "mlstm", "mixer": memory, "mlp": {"kind": "dense", "ff": 352}},
                       {"type": "parallel", "mlp": mlp,
                        "mixer": {"left": left, "right": right, "left_scale": 0.5, "right_scale": 0.5}},
                       {"type": "mlstm", "mixer": memory, "mlp": mlp}]}


def _sebudra_stand_in(vocab_size: int) -> dict:
    """A small model of the Sebudra design: a layer with a windowed attention and a state-space scan side by side over a
    dense feed-forward, a sigmoid-weighted attention over a mixture of experts, a matrix memory with a decay per key
    channel, and the first layer once more with its tensors and a cache of its own."""
    mlp = {"kind": "moe", "router": {"experts": 6, "top": 2, "scale": 2.0, "groups": {"count": 3, "keep": 2}},
           "expert": {"ff": 96}, "shared": {"ff": 128}}
    dense = {"kind": "dense", "ff": 352, "limit": 3.0}
    left = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 32 ** -0.5, "mask": {"size": 48},
            "rot": {"base": 10000.0, "dims": 16, "scaling": {"factor": 4.0, "original": 256, "fast": 16.0, "slow": 1.0}}}
    right = {"heads": 4, "vdim": 32, "state": 16, "groups": 2, "conv": 4, "norm_groups": 2}
    first = {"type": "parallel", "mlp": dense,
             "mixer": {"left": left, "right": right, "left_scale": 0.5, "right_scale": 0.5}}
    return {"architecture": "Sebudra", "vocab": vocab_size, "width": 128, "norm": {"eps": 1e-6},
            "embedding": {"scale": 128 ** 0.5}, "max_position_embeddings": 1024,
            "layers": [first,
                       {"type": "attention", "mlp": mlp,
                        "mixer": {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 32 ** -0.5, "softcap": 20.0,
                                  "rot": {"base": 10000.0, "dims": 32}}},
                       {"type": "gla", "mlp": mlp, "mixer": {"heads": 4, "dim": 32, "vdim": 32, "tau": 8.0, "rank": 8}},
                       dict(first, weights_of=0)]}


def _kofipel_stand_in(vocab_size: int) -> dict:
    """A small model of the Kofipel design: a delta memory, an attention over a window that keeps the first tokens, a delta
    memory without a feed-forward; the last two layers run twice."""
    mlp = {"kind": "dense", "ff": 384}
    memory = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "conv": 4, "decay_rank": 16, "gate_rank": 16}
    attention = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 32 ** -0.5, "softcap": 30.0,
                 "mask": {"size": 48, "keep_first": 8}, "rot": {"base": 10000.0, "dims": 16}}
    return {"architecture": "Kofipel", "vocab": vocab_size, "width": 128, "norm": {"eps": 1e-6}, "canon": {"taps": 3},
            "token_side": {"dim": 16}, "loop": {"start": 1, "stop": 3, "times": 2}, "max_position_embeddings": 1024,
            "layers": [{"type": "channel_delta", "mixer": memory, "mlp": mlp}, {"type": "attention", "mixer": attention, "mlp": mlp},
                       {"type": "channel_delta", "mixer": memory, "mlp": None}]}


def _daferax_stand_in(vocab_size: int) -> dict:
    """A small model of the Daferax design: two attentions whose values mix around a windowed latent attention, mixtures of
    experts chosen within the best groups, the last layer without one."""
    mlp = {"kind": "moe", "router": {"experts": 6, "top": 2, "scale": 2.0, "groups": {"count": 3, "keep": 2}},
           "expert": {"ff": 64}, "shared": {"ff": 160}}
    attention = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 32 ** -0.5, "v_mix": True,
                 "rot": {"base": 10000.0, "dims": 32}}
    latent = {"heads": 4, "dim": 24, "rot_dim": 8, "vdim": 24, "kv_rank": 40, "scale": 32 ** -0.5, "mask": {"size": 48},
              "rot": {"base": 10000.0, "dims": 8, "scaling": {"factor": 4.0, "original": 256, "fast": 16.0, "slow": 1.0}}}
    return {"architecture": "Daferax", "vocab": vocab_size, "width": 128, "norm": {"eps": 1e-6}, "max_position_embeddings": 1024,
            "layers": [{"type": "attention", "mixer": attention, "mlp": mlp}, {"type": "latent_attention", "mixer": latent, "mlp": mlp},
                       {"type": "attention", "mixer": attention, "mlp": None}]}


def tiny_config(vocab_size: int = 260, name: str = "tiny") -> dict:
    """config.json of a random stand-in model."""
    if name == "daferax":
        return _daferax_stand_in(vocab_size)
    if name == "kofipel":
        return _kofipel_stand_in(vocab_size)
    if name == "sebudra":
        return _sebudra_stand_in(vocab_size)
    if name == "tufevik":
        return _tufevik_stand_in(vocab_size)
    if name == "fororax":
        return _fororax_stand_in(vocab_size)
    if name == "givelix":
        return _givelix_stand_in(vocab_size)
    return {"architectures": ["Qwen2ForCausalLM"], "model_type": "qwen2", "attention_bias": True,
            "tie_word_embeddings": True, **RANDOM_MODELS[name], "vocab_size": vocab_size}


class _Runtime:
    """What the subcommands share: the model, a tokenizer if text can be handled, engine settings."""

    def __init__(self, args) -> None:
        import torch

        from .models import load_model, random_model
        from .tokenizer import ByteTokenizer

        if args.device not in ("auto", "cuda") and not args.device.startswith("cuda:"):
            raise SystemExit(f"llmserve: device {args.device!r}: this engine runs on CUDA devices only")
        if not torch.cuda.is_available():
            raise SystemExit("llmserve: no CUDA device; this engine has no CPU path")
        device = "cuda" if args.device == "auto" else args.device
        self.args = args
        if args.model:
            self.model = load_model(args.model, dtype=args.dtype, device=device)
            self.tokenizer = None        # a model folder is served by token ids; text tokenizers are outside this engine
        else:
            self.tokenizer = ByteTokenizer()
            vocab = max(self.tokenizer.vocab_size, RANDOM_MODELS[args.random]["vocab_size"])
            self.model = random_model(tiny_config(vocab, args.random), args.seed, dtype=args.dtype, device=device)

    def engine(self, *, batch_size=None, mode="continuous", policy="fcfs", metrics=False):
        from .config.runtime_config import CacheConfig, SchedulerConfig
        from .engine.llm_engine import LLMEngine

        args = self.args
        return LLMEngine(self.model, self.tokenizer,
                         cache_config=CacheConfig(block_size=args.block_size, num_blocks=args.num_blocks),
                         scheduler_config=SchedulerConfig(max_batch_size=batch_size or args.batch_size,
                                                          max_tokens_per_step=args.max_tokens_per_step, policy=policy),
                         scheduler_mode=mode, prefill_chunk_size=args.prefill_chunk_size,
                         collect_iteration_metrics=metrics)


class NaiveDecoder:
    """The sequential baseline of ``--config naive``: every token recomputes its whole prefix
    (``src/llmserve/engine.py:75-105``), here as one whole-prompt step of the same step function."""

    def __init__(self, model) -> None:
        from .cache.manager import CacheManager
        from .config.runtime_config import CacheConfig
        from .engine.step import StepRunner
        from .models import cache_requirements
        from .sampling.sampler import Sampler

        limit = model.spec.max_position_embeddings
        self.cache = CacheManager(cache_requirements(model.spec), CacheConfig(16, -(-limit // 16)), model.dtype,
                                  model.device, limit, num_state_slots=1)
        self.runner = StepRunner(model, self.cache, limit, 1)
        self.sampler = Sampler(model.vocab_size, 1, model.device)
        self._turn = asyncio.Lock()

    async def generate(self, prompt_token_ids, config, callback=None) -> list[int]:
        from .engine.step import StepEntry

        produced: list[int] = []
        async with self._turn:
            while len(produced) < config.max_new_tokens:
                prefix = [*prompt_token_ids, *produced]
                self.cache.create("naive")
                try:
                    logits = self.runner.run([StepEntry("naive", prefix, [len(prefix) - 1])])
                    token = self.sampler.sample(logits, [config], [len(produced)])[0]
                finally:
                    self.cache.free("naive")
                produced.append(token)
                if callback is not None:
                    callback(token)
                if token in config.stop_token_ids:
                    break
                await asyncio.sleep(0)
        return produced


def run_benchmark(args) -> dict:
    """``llmserve benchmark``: synthetic traffic of the profile against one of four serving set-ups."""
    from .sampling.sampler import GenerationConfig
    from .workload import TrafficProfile, make_traffic, replay_traffic, summarise

    runtime = _Runtime(args)
    model = runtime.model
    profile = TrafficProfile.from_file(args.profile) if args.profile and Path(args.profile).exists() else TrafficProfile()
    overrides = {key: value for key, value in (("requests", args.requests), ("arrival_rate", args.arrival_rate)) if value}
    profile = TrafficProfile(**{**vars(profile), **overrides}).fitted_to(model.vocab_size, model.spec.max_position_embeddings)
    traffic = make_traffic(profile)

    def sampling(item):
        return GenerationConfig(max_new_tokens=item.max_new_tokens, temperature=0.0, seed=args.seed)

    async def drive():
        if args.config == "naive":
            decoder = NaiveDecoder(model)
            return await replay_traffic(f"naive-{args.policy}", traffic, lambda item, on_token: decoder.generate(
                item.prompt_token_ids, sampling(item), on_token)), None
        engine = runtime.engine(batch_size=1 if args.config == "paged" else None, policy=args.policy, metrics=True,
                                mode="static" if args.config == "static" else "continuous")
        async with engine:
            result = await replay_traffic(f"{args.config}-{args.policy}", traffic, lambda item, on_token: engine.generate(
                list(item.prompt_token_ids), sampling(item), on_token, request_id=item.request_id))
            result.cache = engine.cache_stats
            result.extra["engine"] = engine.iteration_stats
        return result, engine

    result, _ = asyncio.run(drive())
    result.extra["profile"] = {**{k: v for k, v in vars(profile).items() if k not in ("prompt", "output")},
                               "prompt": vars(profile.prompt), "output": vars(profile.output)}
    target = Path(args.output)
    target.parent.mkdir(parents=True, exist_ok=True)
    target.write_text(json.dumps(result.as_dict(), indent=2) + "\n")
    summary = summarise(result)
    print(json.dumps(summary, indent=2))
    return summary


def run_generate(args) -> list[dict]:
    """``llmserve generate``: one JSON line per prompt with its ids and the generated ids."""
    from .sampling.sampler import GenerationConfig

    runtime = _Runtime(args)
    prompts = [[int(item) for item in text.replace(",", " ").split()] for text in args.prompt_ids or []]
    for text in args.prompt or []:
        if runtime.tokenizer is None:
            raise SystemExit("llmserve generate: --prompt needs a tokenizer (the random model has one); give --prompt-ids")
        prompts.append(runtime.tokenizer.encode(text))
    if not prompts:
        raise SystemExit("llmserve generate: give --prompt-ids or --prompt")
    sampling = GenerationConfig(max_new_tokens=args.max_new_tokens, temperature=args.temperature, top_p=args.top_p,
                                seed=args.seed, stop_token_ids=tuple(args.stop_token_ids or ()))
    records = []
    for prompt, output in zip(prompts, runtime.engine().generate_many(prompts, sampling)):
        record = {"prompt_ids": prompt, "output_ids": output}
        if runtime.tokenizer is not None:
            record["text"] = runtime.tokenizer.decode(output)
        print(json.dumps(record))
        records.append(record)
    return records


def _engine_options(parser: argparse.ArgumentParser) -> None:
    parser.add_argument("--model", help="folder with config.json and safetensors (default: a random stand-in model)")
    parser.add_argument("--random", choices=sorted(RANDOM_MODELS), default="tiny", help="which random stand-in model")
    parser.add_argument("--device", default="auto")
    parser.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    parser.add_argument("--batch-size", type=int, default=16)
    parser.add_argument("--block-size", type=int, default=16)
    parser.add_argument("--num-blocks", type=int, default=1024)
    parser.add_argument("--prefill-chunk-size", type=int, default=2048)
    parser.add_argument("--max-tokens-per-step", type=int, default=2048)
    parser.add_argument("--seed", type=int, default=7)


def build_parser() -> argparse.ArgumentParser:
    parser = argparse.ArgumentParser(prog="llmserve")
    commands = parser.add_subparsers(dest="command", required=True)
    benchmark = commands.add_parser("benchmark", help="synthetic traffic against the engine; latency and throughput report")
    benchmark.add_argument("--config", choices=("naive", "paged", "static", "continuous"), default="continuous")
    benchmark.add_argument("--policy", choices=("fcfs", "sjf", "priority"), default="fcfs")
    benchmark.add_argument("--profile", default="configs/benchmark-sharegpt.yaml")
    benchmark.add_argument("--requests", type=int)
    benchmark.add_argument("--arrival-rate", type=float)
    benchmark.add_argument("--output", default="artifacts/benchmark.json")
    _engine_options(benchmark)
    generate = commands.add_parser("generate", help="generate token ids for given prompts")
    generate.add_argument("--prompt-ids", action="append", help="token ids, separated by spaces or commas")
    generate.add_argument("--prompt", action="append", help="text (needs a tokenizer)")
    generate.add_argument("--max-new-tokens", type=int, default=32)
    generate.add_argument("--temperature", type=float, default=0.0)
    generate.add_argument("--top-p", type=float, default=1.0)
    generate.add_argument("--stop-token-ids", type=int, nargs="*")
    _engine_options(generate)
    replay = commands.add_parser("replay", help="trace replay: steps of token ids from standard input, logits to files "
                                                "(the same program as bin/trace_run)")
    replay.description = "every option after `replay` goes to trace_run: --model --dtype --out --max-tokens"
    return parser


def parse(argv=None):
    """Arguments of the command line; ``rest`` holds what follows ``replay`` (trace_run's own options)."""
    parser = build_parser()
    args, rest = parser.parse_known_args(argv)
    if rest and args.command != "replay":
        parser.error("unrecognized arguments: " + " ".join(rest))
    args.rest = rest
    return args


def main(argv=None) -> int:
    args = parse(argv)
    if args.command == "benchmark":
        run_benchmark(args)
    elif args.command == "generate":
        run_generate(args)
    else:
        from .engine.trace_replay import main as replay_main
        return replay_main(args.rest)
    return 0


if __name__ == "__main__":
    sys.exit(main())
