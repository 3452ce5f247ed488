"""The Kofipel design through the engine against the plain implementation (``tests/plain/kofipel_plain.py``): both mixers
alone and together, looped layers, whole prompts, decoding through pages, windows and states, portions down to two tokens,
mixed batches with pages and slots that are used again, other sizes, both precisions, greedy generation through
``LLMEngine``; and the kernels of its mechanisms alone, with inputs made so that a lost key, a window that is one token off,
a sink that is left out, a row of a convolution or a state that is not carried shows."""
import json
import random
import tempfile
from pathlib import Path
from types import SimpleNamespace

import pytest
import torch

import helpers
from plain import kofipel_plain as plain

pytestmark = pytest.mark.gpu


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def attention(heads=4, kv_heads=2, dim=16, window=11, keep_first=3, scale=None, softcap=6.0, rot_dims=8, base=10000.0,
              mlp="default"):
    return {"type": "attention", "mlp": dense() if mlp == "default" else mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "softcap": softcap,
                      "scale": scale if scale is not None else 1.5 / dim ** 0.5,
                      "mask": {"size": window, "keep_first": keep_first}, "rot": {"base": base, "dims": rot_dims}}}


def memory(heads=4, kv_heads=2, dim=16, vdim=24, conv=3, decay_rank=5, gate_rank=7, mlp="default"):
    return {"type": "channel_delta", "mlp": dense() if mlp == "default" else mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank,
                      "gate_rank": gate_rank}}


def model(layers, width=64, vocab=211, taps=3, side=10, loop=(0, 0, 1), eps=1e-5, positions=2048):
    return {"architecture": "Kofipel", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "canon": {"taps": taps}, "token_side": {"dim": side}, "max_position_embeddings": positions,
            "loop": dict(zip(("start", "stop", "times"), loop))}


CONFIGS = {
    "attention_only": model([attention(), attention(heads=6, kv_heads=6, dim=8, window=5, keep_first=0, rot_dims=2, mlp=None),
                             attention(heads=2, kv_heads=1, dim=32, window=64, keep_first=17, rot_dims=32, softcap=1.5)]),
    "memory_only": model([memory(), memory(heads=2, kv_heads=2, dim=32, vdim=32, conv=4, mlp=None),
                          memory(heads=6, kv_heads=1, dim=8, vdim=16, conv=2)], taps=2),
    # both kinds, a range of layers run three times (an attention layer's pages once per pass among them)
    "all_kinds": model([attention(), memory(), attention(window=30, keep_first=9, mlp=None), memory(heads=2, kv_heads=1, dim=64, vdim=16),
                        attention(heads=2, kv_heads=2)], width=80, taps=4, loop=(1, 3, 3)),
    # the whole model twice, from its first layer on
    "loop_from_the_start": model([memory(mlp=None), attention(window=7, keep_first=1)], taps=4, loop=(0, 2, 2)),
    # head sizes that the tensor-core kernels take in bfloat16, and widths beyond one piece of four channels a thread
    "tensor_core_sizes": model([memory(heads=6, kv_heads=3, dim=64, vdim=80, conv=4, decay_rank=16, gate_rank=32),
                                attention(heads=4, kv_heads=2, dim=64, window=100, keep_first=5, rot_dims=32),
                                memory(heads=2, kv_heads=1, dim=128, vdim=128, conv=4),
                                attention(heads=3, kv_heads=1, dim=96, window=70, keep_first=65, rot_dims=96)], width=160, taps=4, side=32),
    # values that many models make equal or one: one head, a window of one token, one kept token, no rotated pair but one,
    # one tap everywhere, ranks of one, a side input of one number, a cap that caps nothing, a scale of one
    "equal_or_one": model([attention(heads=1, kv_heads=1, dim=32, window=1, keep_first=1, scale=1.0, softcap=1000.0, rot_dims=2),
                           memory(heads=1, kv_heads=1, dim=32, vdim=32, conv=1, decay_rank=1, gate_rank=1),
                           attention(heads=3, kv_heads=3, dim=16, window=4096, keep_first=2, rot_dims=16, mlp=dense(64)),
                           memory(heads=1, kv_heads=1, dim=1, vdim=1, conv=1, decay_rank=1, gate_rank=1, mlp=None)],
                          width=64, taps=1, side=1, loop=(3, 4, 1)),
    # sizes that no vector load or few-rows product takes; nine query heads on three; more taps than the fused kernels
    # were built for; a kept range that is longer than the window and ends inside a page; memory heads wider than 128
    "odd_sizes": model([attention(heads=9, kv_heads=3, dim=20, window=23, keep_first=37, rot_dims=6),
                        memory(heads=5, kv_heads=5, dim=12, vdim=28, conv=6, decay_rank=3, gate_rank=9, mlp=None),
                        attention(heads=5, kv_heads=1, dim=12, window=7, keep_first=4, rot_dims=12, base=77.0, softcap=2.5, mlp=dense(50)),
                        memory(heads=3, kv_heads=1, dim=140, vdim=5, conv=5, mlp=dense(34))], width=102, vocab=333, taps=6, side=7,
                       loop=(2, 4, 2)),
    # a width beyond what a thread's piece covers at once, and taps that the fused kernel takes
    "wide": model([memory(heads=2, kv_heads=1, dim=40, vdim=24), attention(window=19, keep_first=2)], width=2100, vocab=97, taps=3,
                  side=20),
}
# float32: the recurrences pass rounding on from token to token.  A lost key, a window that is one token off or a state
# that is not carried moves a row by a hundredth and more.
RMS_LIMIT = {"float32": 2.0e-4, "bfloat16": 8.0e-2}
# A side input of one number passes a norm, and a key of one channel becomes a unit vector: only their signs are left, and a
# value near zero falls either way under bfloat16 rounding.  That model is compared in float32.
CASES = [(name, dtype) for name in sorted(CONFIGS) for dtype in ("float32", "bfloat16") if (name, dtype) != ("equal_or_one", "bfloat16")]
_MODELS: dict = {}


def folder_of(name: str):
    if name not in _MODELS:
        holder = tempfile.TemporaryDirectory(prefix=f"kofipel_{name}_")
        plain.write_model(holder.name, CONFIGS[name], seed=83 + len(_MODELS))
        _MODELS[name] = (holder, Path(holder.name), plain.load_folder(holder.name))
    return _MODELS[name][1]


def reference(name: str, tokens):
    folder_of(name)
    config, weights = _MODELS[name][2]
    return plain.forward_full(config, weights, tokens).to(torch.float32)


def replay(name: str, dtype: str, steps, max_tokens: int, page: int = 16, max_requests: int = 4):
    from llm_serving_engine_b200.engine.trace_replay import replay as run

    with tempfile.TemporaryDirectory(prefix="kofipel_out_") as out:
        run(folder_of(name), dtype, out, max_tokens, [json.dumps(step) for step in steps], block_size=page,
            max_requests=max_requests)
        return helpers.collect(steps, Path(out))


def compare(name, dtype, requests, got, what):
    """Row error over logit size, every row within the limit."""
    for rid, tokens in requests.items():
        want = reference(name, tokens)
        assert got[rid].shape == want.shape, f"{what}: {rid}: shape {tuple(got[rid].shape)} against {tuple(want.shape)}"
        centred = want - want.mean(-1, keepdim=True)
        per_row = (got[rid] - want).double().pow(2).mean(-1).sqrt() / centred.double().pow(2).mean().sqrt()
        worst = float(per_row.max())
        assert worst <= RMS_LIMIT[dtype], (f"{what}: {name} {dtype} request {rid}: row error / logit size {worst:.2e} at position "
                                           f"{int(per_row.argmax())}, first above the limit {int((per_row > RMS_LIMIT[dtype]).nonzero()[0])}")


def some_requests(name, lengths, seed=5):
    rng = random.Random(seed)
    vocab = CONFIGS[name]["vocab"]
    return {f"r{index}": helpers.random_tokens(rng, vocab, length) for index, length in enumerate(lengths)}


# ------------------------------------------------------------------ through the engine
@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_prompts(name, dtype):
    requests = some_requests(name, [1, 2, 17, 70])
    got = replay(name, dtype, helpers.trace_whole(requests), helpers.max_tokens_for(requests))
    compare(name, dtype, requests, got, "whole")


@pytest.mark.parametrize("name", ["all_kinds", "odd_sizes", "equal_or_one", "loop_from_the_start", "wide"])
def test_every_layer_against_the_plain_layers(name):
    """The float32 residual after every layer run, through the engine's own step function."""
    from llm_serving_engine_b200.cache.manager import CacheManager
    from llm_serving_engine_b200.config import CacheConfig
    from llm_serving_engine_b200.engine.step import StepEntry, StepRunner
    from llm_serving_engine_b200.models import cache_requirements, load_model
    from llm_serving_engine_b200.parts.linear import reduce_partials

    tokens = some_requests(name, [45], seed=2)["r0"]
    engine_model = load_model(folder_of(name), dtype="float32")
    cache = CacheManager(cache_requirements(engine_model.spec), CacheConfig(block_size=8, num_blocks=16), engine_model.dtype,
                         engine_model.device, engine_model.spec.max_position_embeddings, num_state_slots=2)
    runner = StepRunner(engine_model, cache, 64, 2, use_graphs=False)
    seen = []

    def after_layer(position, stream):
        """A layer's output is still pending with its norm (the next layer's norm applies both): add it to a copy."""
        pending = plain.rms(reduce_partials(stream.delta).double(), stream.delta_norm.eps) * stream.delta_norm.weight.double()
        seen.append((stream.residual.double() + pending).cpu())

    engine_model.layer_hook = after_layer
    cache.create("a")
    runner.run([StepEntry("a", tokens, [])])
    config, weights = _MODELS[name][2]
    want = plain.forward_layers(config, weights, tokens)[1:]
    assert len(seen) == len(want)
    for index, (got, expected) in enumerate(zip(seen, want)):
        assert float((got - expected).abs().max()) <= 5e-5 * float(expected.abs().max()), f"layer run {index}"


@pytest.mark.parametrize("name,dtype", CASES)
def test_prompt_then_token_by_token(name, dtype):
    """Decoding reads the pages, windows and states that the prompt step left (single tokens are replayed from a
    captured graph); a prompt of one token and of fewer tokens than a convolution has taps are among them, and the
    attention windows pass over decoded tokens and come away from the kept first tokens."""
    requests = some_requests(name, [60, 9, 3, 25], seed=6)
    got = replay(name, dtype, helpers.trace_tail_decode(requests, tail=24), helpers.max_tokens_for(requests))
    compare(name, dtype, requests, got, "tail decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["all_kinds", "odd_sizes", "tensor_core_sizes"])
def test_portions_of_changing_size(name, dtype):
    """Portions shorter than the convolutions' windows and than the attention windows, portions that end on a page's
    and a chunk's border, one token at a time between longer ones."""
    requests = some_requests(name, [150, 33], seed=7)
    for sizes in ((7, 2, 13, 3, 2, 31, 5, 16, 2, 64, 17), (2,), (16, 16, 1, 15, 17), (1, 2, 3, 1, 1, 64, 63)):
        got = replay(name, dtype, helpers.trace_portions(requests, sizes), helpers.max_tokens_for(requests))
        compare(name, dtype, requests, got, f"portions {sizes}")


@pytest.mark.parametrize("name,dtype", [("all_kinds", "float32"), ("memory_only", "float32"), ("odd_sizes", "float32"),
                                        ("tensor_core_sizes", "bfloat16"), ("tensor_core_sizes", "float32")])
def test_a_long_prompt_whole_and_in_portions_that_cut_chunks_anywhere(name, dtype):
    requests = some_requests(name, [413], seed=13)
    whole = replay(name, dtype, helpers.trace_whole(requests), 448)
    compare(name, dtype, requests, whole, "long whole")
    cut = replay(name, dtype, helpers.trace_portions(requests, (130, 1, 199, 17, 65, 2)), 448)
    compare(name, dtype, requests, cut, "long in portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("page", [16, 8])
def test_mixed_batches_reuse_pages_and_slots(dtype, page):
    """Nine requests through four slots and a pool sized for the live ones only: a page's old rows must not be read (the
    windowed layers give pages back while a request runs, all but those of the kept first tokens), and a slot's states
    and windows must start from zero for the request that takes it next."""
    requests = some_requests("all_kinds", [61, 5, 90, 33, 2, 47, 130, 18, 64], seed=8)
    steps, peak = helpers.trace_mixed(requests, seed=3, max_live=4)
    got = replay("all_kinds", dtype, steps, peak, page=page)
    compare("all_kinds", dtype, requests, got, "mixed")


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_long_portions_beside_single_tokens(dtype):
    """Steps in which portions of many rows (delta memory in chunks), of few rows (row by row) and single decoded tokens
    stand beside one another; pages and slots are used again by a fourth request."""
    name = "tensor_core_sizes"
    requests = some_requests(name, [156, 150, 270, 140], seed=21)
    a, b, c, d = (requests[f"r{index}"] for index in range(4))

    def entry(rid, tokens, first, count):
        return {"id": rid, "tokens": tokens[first:first + count], "want": list(range(count))}

    steps = [
        {"step": 0, "entries": [entry("r0", a, 0, 150), entry("r1", b, 0, 3)], "end": []},
        {"step": 1, "entries": [entry("r0", a, 150, 1), entry("r1", b, 3, 140), entry("r2", c, 0, 130)], "end": []},
        {"step": 2, "entries": [entry("r0", a, 151, 1), entry("r1", b, 143, 1), entry("r2", c, 130, 135)], "end": []},
        {"step": 3, "entries": [entry("r0", a, 152, 4), entry("r1", b, 144, 6), entry("r2", c, 265, 1)], "end": ["r0", "r1"]},
        {"step": 4, "entries": [entry("r2", c, 266, 1), entry("r3", d, 0, 128)], "end": []},
        {"step": 5, "entries": [entry("r2", c, 267, 3), entry("r3", d, 128, 12)], "end": ["r2", "r3"]},
    ]
    got = replay(name, dtype, steps, 640)
    compare(name, dtype, requests, got, "long portions beside single tokens")


def test_a_batch_gives_what_each_request_gives_alone():
    for name in ("all_kinds", "odd_sizes"):
        requests = some_requests(name, [37, 12, 80, 5], seed=9)
        steps, peak = helpers.trace_mixed(requests, seed=4, max_live=4)
        together = replay(name, "float32", steps, peak)
        for rid, tokens in requests.items():
            alone = replay(name, "float32", helpers.trace_whole({rid: tokens}), helpers.max_tokens_for({rid: tokens}))
            assert float((together[rid] - alone[rid]).abs().max()) <= 2e-5 * float(alone[rid].abs().max())


def test_long_decoding_crosses_key_chunks_and_many_pages():
    """600 single tokens after a short prompt: the windows slide over hundreds of decoded tokens far from the kept first
    ones, many pages are given back and taken again, and the recurrent states are carried six hundred times."""
    requests = some_requests("all_kinds", [610], seed=10)
    got = replay("all_kinds", "float32", helpers.trace_tail_decode(requests, tail=600), 640)
    compare("all_kinds", "float32", requests, got, "long decoding")


def test_greedy_generation_through_the_engine_and_its_scheduler():
    """More requests than the scheduler keeps live, prompts cut into portions: every request's greedy tokens equal
    the plain implementation's (float32; a request whose top two logits are closer than the arithmetic's noise is
    skipped from that token on)."""
    from llm_serving_engine_b200.config import CacheConfig, SchedulerConfig
    from llm_serving_engine_b200.engine.llm_engine import LLMEngine
    from llm_serving_engine_b200.models import load_model
    from llm_serving_engine_b200.sampling.sampler import GenerationConfig

    name = "all_kinds"
    engine = LLMEngine(load_model(folder_of(name), dtype="float32"), None,
                       cache_config=CacheConfig(block_size=16, num_blocks=40),
                       scheduler_config=SchedulerConfig(max_batch_size=3, max_tokens_per_step=48), prefill_chunk_size=20)
    prompts = list(some_requests(name, [30, 7, 55, 2, 19, 41], seed=12).values())
    new_tokens = 12
    produced = engine.generate_many(prompts, GenerationConfig(max_new_tokens=new_tokens, temperature=0.0))
    for prompt, tokens in zip(prompts, produced):
        assert len(tokens) == new_tokens
        logits = reference(name, prompt + tokens)
        for index, token in enumerate(tokens):
            row = logits[len(prompt) + index - 1]
            top = torch.topk(row, 2).values
            if float(top[0] - top[1]) < 1e-3 * float(row.abs().max()):
                break
            assert int(row.argmax()) == token, f"token {index} of a {len(prompt)}-token prompt"


def _drawn_model(rng):
    """One to five layers of both kinds in any order with sizes drawn one by one, a range of them looped."""
    layers = []
    for _ in range(rng.randint(1, 5)):
        mlp = None if rng.random() < 0.2 else dense(rng.choice([24, 50, 88, 128]))
        kv_heads, group = rng.choice([1, 2, 3]), rng.choice([1, 2, 4])
        if rng.random() < 0.5:
            dim = rng.choice([16, 24, 32, 48, 64, 96, 128])
            layers.append(attention(kv_heads * group, kv_heads, dim, window=rng.choice([1, 3, 16, 17, 33, 64, 100, 500]),
                                    keep_first=rng.choice([0, 1, 4, 16, 17, 40]), scale=rng.choice([1.0, 1.5, 2.0]) / dim ** 0.5,
                                    softcap=rng.choice([1.0, 5.0, 20.0, 100.0]), base=rng.choice([100.0, 10000.0, 1000000.0]),
                                    rot_dims=rng.choice([d for d in (2, 4, 8, dim // 2, dim) if d % 2 == 0]), mlp=mlp))
        else:
            layers.append(memory(kv_heads * group, kv_heads, rng.choice([4, 16, 32, 64, 96, 160]), rng.choice([8, 24, 64, 100]),
                                 rng.choice([1, 2, 3, 4, 5]), rng.choice([1, 4, 16, 24]), rng.choice([2, 8, 20]), mlp))
    start = rng.randint(0, len(layers) - 1)
    return model(layers, width=rng.choice([48, 64, 90, 120, 256]), vocab=rng.choice([97, 300, 501]), taps=rng.choice([1, 2, 3, 4, 5]),
                 side=rng.choice([3, 8, 16, 40]), loop=(start, rng.randint(start, len(layers)), rng.choice([1, 2, 3])),
                 eps=rng.choice([1e-5, 1e-6]))


@pytest.mark.parametrize("seed", range(10))
def test_architectures_drawn_at_random(seed):
    """Kinds, order, sizes, constants and loops drawn at random, four requests whole, in portions of drawn sizes, with
    decoded tails and in mixed batches through four slots, in float32 against the plain implementation."""
    rng = random.Random(2000 + seed)
    config = _drawn_model(rng)
    name = f"drawn_{seed}"
    CONFIGS[name] = config
    try:
        requests = {f"r{index}": helpers.random_tokens(rng, config["vocab"], count)
                    for index, count in enumerate([rng.randint(1, 40), rng.randint(100, 300), rng.randint(30, 150), rng.randint(2, 70)])}
        sizes = tuple(rng.choice([1, 2, 3, 7, 16, 33, 64, 130]) for _ in range(6))
        peak = helpers.max_tokens_for(requests)
        compare(name, "float32", requests, replay(name, "float32", helpers.trace_whole(requests), peak), f"whole {config['layers']}")
        compare(name, "float32", requests, replay(name, "float32", helpers.trace_portions(requests, sizes), peak), f"portions {sizes}")
        compare(name, "float32", requests, replay(name, "float32", helpers.trace_tail_decode(requests, tail=20), peak), "tail decoded")
        steps, live = helpers.trace_mixed(requests, seed=seed, max_live=4)
        compare(name, "float32", requests, replay(name, "float32", steps, live), "mixed")
    finally:
        CONFIGS.pop(name, None)
        _MODELS.pop(name, None)


# ------------------------------------------------------------------ the mechanisms' kernels alone
def _step(lengths, first_positions=None, slots=None):
    """The step's tensors that the kernels read, for requests of ``lengths`` rows laid one after the other."""
    first_positions = first_positions or [0] * len(lengths)
    slots = slots if slots is not None else list(range(len(lengths)))
    seg, pos, start = [], [], [0]
    for index, (count, first) in enumerate(zip(lengths, first_positions)):
        seg += [index] * count
        pos += list(range(first, first + count))
        start.append(start[-1] + count)
    as_int = lambda values: torch.tensor(values, dtype=torch.int32, device="cuda")
    return SimpleNamespace(segment_of_token=as_int(seg), positions=as_int(pos), segment_start=as_int(start),
                           segment_first_position=as_int(first_positions), segment_state_slot=as_int(slots),
                           decode_only=all(count == 1 for count in lengths))


def _cuts(total, sizes):
    """(first row, rows) of the portions of ``sizes``, repeated until ``total`` rows are spent."""
    out, at, index = [], 0, 0
    while at < total:
        size = min(sizes[index % len(sizes)], total - at)
        out.append((at, size))
        at, index = at + size, index + 1
    return out


def _paged(q, k, v, cuts, page, dtype, scale, window, keep_first, cap):
    """q [T, H, d], k and v [T, G, d] of one request through the paged attention in the portions ``cuts``.  Keys and values
    are written to pages scattered in a pool whose other rows hold NaN; before every portion the pages that no row of it
    may read are overwritten with NaN and their table entries point nowhere."""
    from llm_serving_engine_b200.kernels import ops

    total, n_q, d = q.shape
    n_kv, pages = k.shape[1], -(-total // page)
    order = torch.randperm(pages + 4, generator=torch.Generator().manual_seed(total + page))[:pages].to(torch.int32)
    keys = torch.full((pages + 4, n_kv, page, d), float("nan"), dtype=dtype, device="cuda")
    values = torch.full_like(keys, float("nan"))
    table = order.clone()
    sink = torch.zeros(n_q, device="cuda")
    out = []
    for at, count in cuts:
        step = _step([count], [at])
        for logical in range(-(-keep_first // page), (at - window + 1) // page if at - window + 1 > 0 else 0):
            if int(table[logical]) >= 0:
                keys[int(table[logical])] = values[int(table[logical])] = float("nan")
                table[logical] = -1
        places = torch.arange(at, at + count)
        where, offset = order[places // page].long().cuda(), (places % page).cuda()
        keys[where, :, offset] = k[at:at + count].to(dtype).cuda()
        values[where, :, offset] = v[at:at + count].to(dtype).cuda()
        attended = torch.empty(count, n_q, d, dtype=dtype, device="cuda")
        ops.attention_scored(q[at:at + count].to(dtype).cuda().contiguous(), keys, values, attended, table.view(1, -1).cuda(),
                             step.segment_of_token, step.positions, scale, sink=sink, segment_start=step.segment_start,
                             segment_first_position=step.segment_first_position, window=window, cap=cap, keep_first=keep_first)
        out.append(attended.float().cpu())
    return torch.cat(out)


def _plain_attention(q, k, v, scale, window, keep_first, cap):
    total, heads = q.shape[0], q.shape[1]
    k, v = (t.double().repeat_interleave(heads // t.shape[1], dim=1) for t in (k, v))
    scores = torch.einsum("ihd,jhd->hij", q.double(), k) * scale
    scores = cap * torch.tanh(scores / cap)
    weights = plain.sink_softmax(scores.masked_fill(~plain.visible(total, window, keep_first), float("-inf")))
    return torch.einsum("hij,jhe->ihe", weights, v)


# head sizes that the general kernel takes and that the tensor-core kernel takes in bfloat16
_HEADS = [(4, 2, 24), (4, 2, 64), (6, 2, 48), (8, 1, 128), (3, 1, 32)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads", _HEADS)
@pytest.mark.parametrize("window,keep_first", [(1, 1), (7, 3), (40, 16), (40, 17), (64, 0), (256, 63), (20, 300), (100, 64)])
def test_a_window_that_keeps_the_first_keys(dtype, heads, window, keep_first):
    """One key far stronger than the others just inside and just outside the last row's window, and among and just behind
    the kept first keys; pages between the two ranges hold NaN once no row may read them.  Rows come whole, as a prompt
    and a single token, in portions of two and of changing size."""
    torch.manual_seed(17)
    (n_q, n_kv, d), context, page, cap = heads, 390, 16, 9.0
    scale = 1.5 / d ** 0.5
    last = context - 1
    places = {last - window + 1, last - window, keep_first - 1, keep_first, keep_first + 1, 0, last, 255, 256}
    for special in sorted(place for place in places if 0 <= place <= last):
        q, k, v = (torch.randn(context, n, d).to(dtype).float() for n in (n_q, n_kv, n_kv))
        k[special, 0] = 3.0 * q[last, 1]        # head 1 of the last row finds it, if it may
        v[special, 0] = 5.0
        want = _plain_attention(q, k, v, scale, window, keep_first, cap)
        inside = last - special < window or special < keep_first
        assert (float(want[-1, 1].mean()) > 2.5) == inside
        every = [[(0, context)], [(0, last), (last, 1)]]
        if special in (keep_first, last - window):
            every += [_cuts(context, (2,)) if dtype == torch.bfloat16 else [(0, 300)] + [(300 + a, n) for a, n in _cuts(90, (2,))],
                      _cuts(context, (7, 64, 1, 31, 130, 3))]
        for cuts in every:
            got = _paged(q, k, v, cuts, page, dtype, scale, window, keep_first, cap)
            limit = 3e-5 if dtype == torch.float32 else 3e-2
            error = (got.double() - want).abs()
            assert float(error.max()) <= limit * max(1.0, float(want.abs().max())), (special, len(cuts), int(error.amax((1, 2)).argmax()))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_unit_in_the_denominator(dtype):
    """Rows whose scores are all very low give almost nothing (a softmax without the unit would give the values' mean)."""
    torch.manual_seed(18)
    n_q, n_kv, d, context = 4, 2, 64, 40
    q = torch.randn(context, n_q, d).to(dtype).float()
    direction = torch.randn(d)
    q[:, 2] = direction.to(dtype).float()
    k = torch.randn(context, n_kv, d).to(dtype).float()
    k[:, 1] = (-direction).to(dtype).float()          # head 2's scores: about -cap
    v = torch.ones(context, n_kv, d)
    want = _plain_attention(q, k, v, 1.0, 16, 2, 8.0)
    assert float(want[:, 2].max()) < 0.02 and float(want[:, 0].mean()) > 0.3
    for cuts in ([(0, context)], _cuts(context, (3, 1))):
        got = _paged(q, k, v, cuts, 8, dtype, 1.0, 16, 2, 8.0)
        assert float((got.double() - want).abs().max()) <= (2e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("stacked", [False, True])
@pytest.mark.parametrize("n_q,n_kv,d,rot", [(4, 2, 24, 10), (3, 3, 16, 16), (4, 1, 64, 0), (2, 1, 128, 64)])
def test_rotated_heads_with_factors_and_values_that_are_keys(dtype, stacked, n_q, n_kv, d, rot):
    from llm_serving_engine_b200.kernels import ops

    torch.manual_seed(19)
    rows, page, first, pad = 5, 8, 4001, 3
    width = (n_q + n_kv) * d
    whole = torch.randn(rows, width + pad)
    proj = torch.stack([whole * 0.25, whole * 0.75]) if stacked else whole.to(dtype)
    seen = proj.double().sum(0) if stacked else proj.double()
    bias, factor = torch.randn(width), torch.rand(n_q) * 2 - 0.5
    freq = torch.tensor([3000.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
    positions = torch.arange(first, first + rows, dtype=torch.int32)
    slots = torch.tensor([3, 17, -1, 30, 8], dtype=torch.int32)          # one padding row
    keys = torch.zeros(4, n_kv, page, d, dtype=dtype, device="cuda")
    values, q = torch.zeros_like(keys), torch.zeros(rows, n_q, d, dtype=dtype, device="cuda")
    ops.head_norm_rope_kv_write(proj.cuda(), bias.cuda(), None, None, 1e-5, slots.cuda(), positions.cuda(), freq.cuda(), 1.0, q, keys,
                                values, n_q, n_kv, d, d, q_factor=factor.cuda(), values_are_keys=True)
    heads = (seen[:, :width] + bias.double()).view(rows, n_q + n_kv, d)
    angle = positions.double()[:, None] * freq[None]
    c, s, half = torch.cos(angle)[:, None], torch.sin(angle)[:, None], rot // 2
    a, b = heads[..., :half], heads[..., half:rot]
    turned = torch.cat([a * c - b * s, b * c + a * s, heads[..., rot:]], dim=-1)
    limit = 2e-5 if dtype == torch.float32 else 3e-2
    for row, slot in enumerate(slots.tolist()):
        if slot < 0:
            continue
        assert float((q[row].cpu().double() - turned[row, :n_q] * factor.double()[:, None]).abs().max()) <= limit
        assert float((keys[slot // page, :, slot % page].cpu().double() - turned[row, n_q:]).abs().max()) <= limit
        assert float((values[slot // page, :, slot % page].cpu().double() - heads[row, n_q:]).abs().max()) <= limit
    held = {slot for slot in slots.tolist() if slot >= 0}
    for slot in range(4 * page):
        if slot not in held:
            assert float(keys[slot // page, :, slot % page].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden,taps", [(64, 1), (64, 4), (132, 2), (1028, 3), (2052, 4), (4100, 2), (50, 3), (64, 6)])
@pytest.mark.parametrize("pending", ["none", "plain", "bias", "norm", "stack"])
def test_sum_norm_and_convolution(dtype, hidden, taps, pending):
    """Two requests' rows in portions of changing size beside one another, then single tokens: the pending output's sum (with
    a bias, with a norm of its own, as a stack of partial sums), the norm, and h + conv(h) against the whole sequences; the
    windows at the end hold each request's last rows of h."""
    from llm_serving_engine_b200.kernels import ops

    torch.manual_seed(20)
    lengths, eps = (39, 24), 1e-5
    x = [torch.randn(n, hidden) * 3 for n in lengths]
    delta = [torch.randn(n, hidden).to(torch.float32 if pending == "stack" else dtype) for n in lengths]
    bias, weight, after = torch.randn(hidden), 1 + 0.3 * torch.randn(hidden), torch.rand(hidden) + 0.5
    conv = torch.randn(hidden, taps) * 0.5
    want_x, want, last = [], [], []
    for rows, add in zip(x, delta):
        total = rows.double()
        if pending in ("plain", "stack"):
            total = total + add.double()
        elif pending == "bias":
            total = total + add.double() + bias.double()
        elif pending == "norm":
            total = total + plain.rms(add.double(), 1e-6) * after.double()
        h = plain.rms(total, eps) * weight.double()
        want_x.append(total)
        want.append(h + plain.causal_conv(h, conv.double()))
        last.append(torch.cat([torch.zeros(taps - 1, hidden, dtype=torch.float64), h])[h.shape[0]:])
    state = torch.zeros(3, taps - 1, hidden, device="cuda")
    slots, at, got, got_x = (2, 0), [0, 0], [[], []], [[], []]
    for portions in ((7, 3), (1, 2), (2, 1), (17, 16), (9, 1), (1, 1), (1, 0), (1, 0)):
        live = [i for i in range(2) if portions[i]]
        lens = [portions[i] for i in live]
        step = _step(lens, slots=[slots[i] for i in live])
        take = lambda source: torch.cat([source[i][at[i]:at[i] + portions[i]] for i in live])
        residual, pend = take(x).cuda(), take(delta).cuda()
        if pending == "stack":
            pend = torch.stack([pend * 0.5, pend * 0.25, pend * 0.25])
        out = torch.empty(sum(lens), hidden, dtype=dtype, device="cuda")
        ops.conv_norm(residual, None if pending == "none" else pend.contiguous(), bias.cuda() if pending == "bias" else None,
                      (after.cuda(), 1e-6) if pending == "norm" else None, weight.cuda(), eps, conv.cuda(), state, step, out)
        for i, rows, res in zip(live, out.cpu().double().split(lens), residual.cpu().double().split(lens)):
            got[i].append(rows)
            got_x[i].append(res)
            at[i] += portions[i]
    assert tuple(at) == lengths
    limit = 3e-6 if dtype == torch.float32 else 1e-2
    for i in range(2):
        assert float((torch.cat(got_x[i]) - want_x[i]).abs().max()) <= 3e-6 * float(want_x[i].abs().max())
        assert float((torch.cat(got[i]) - want[i]).abs().max()) <= limit * float(want[i].abs().max())
        if taps > 1:
            assert float((state[slots[i]].cpu().double() - last[i]).abs().max()) <= 3e-6 * float(last[i].abs().max())
    if taps > 1:
        assert float(state[1].abs().max()) == 0.0        # a slot that no request holds


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_last_norm_over_gathered_rows_and_a_settled_residual(dtype):
    from llm_serving_engine_b200.kernels import ops

    torch.manual_seed(22)
    for tokens, hidden in ((9, 64), (5, 50), (3, 11000)):
        x, add = torch.randn(tokens, hidden), torch.randn(tokens, hidden).to(dtype)
        bias, after, weight = torch.randn(hidden), torch.rand(hidden), torch.rand(hidden) + 0.5
        total = x.double() + plain.rms(add.double(), 1e-5) * after.double()
        rows = torch.tensor([tokens - 1, 0, 2], dtype=torch.int32)
        residual, out = x.cuda(), torch.empty(3, hidden, dtype=dtype, device="cuda")
        ops.delta_norm_rmsnorm(residual, add.cuda(), None, (after.cuda(), 1e-5), weight.cuda(), 1e-6, out, rows=rows.cuda(),
                               write_residual=False)
        want = (plain.rms(total, 1e-6) * weight.double())[rows.long()]
        assert float((out.cpu().double() - want).abs().max()) <= (3e-6 if dtype == torch.float32 else 1e-2) * float(want.abs().max())
        assert torch.equal(residual.cpu(), x)
        copy = torch.empty(tokens, hidden, dtype=dtype, device="cuda")
        ops.residual_settle(residual, add.cuda(), bias.cuda(), copy)
        want = x.double() + add.double() + bias.double()
        assert float((residual.cpu().double() - want).abs().max()) <= 1e-6 * float(want.abs().max())
        assert torch.equal(copy, residual.to(dtype))
        table = torch.randn(13, hidden).to(dtype)
        ids = torch.randint(0, 13, (tokens,), dtype=torch.int32)
        before = residual.clone()
        ops.embedding_add(table.cuda(), ids.cuda(), residual)
        assert torch.equal(residual.cpu(), before.cpu() + table[ids.long()].float())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_token_gate_reads_the_layers_part_of_the_table(dtype):
    from llm_serving_engine_b200.kernels import ops

    torch.manual_seed(23)
    for dim, padded, offset, stacked in ((10, 16, 20, False), (24, 32, 0, True), (1, 16, 3, False)):
        rows, vocab = 7, 19
        z = torch.randn(rows, padded) * 2
        given = torch.stack([z * 0.5, z * 0.5]).cuda() if stacked else z.to(dtype).cuda()
        seen = z.double() if stacked else z.to(dtype).double()
        table = torch.randn(vocab, offset + dim + 5).to(dtype)
        ids = torch.randint(0, vocab, (rows,), dtype=torch.int32)
        out = torch.full((rows, padded), float("nan"), dtype=dtype, device="cuda")
        ops.token_gate(given, table.cuda(), offset, ids.cuda(), out, dim)
        want = plain.gelu_tanh(seen[:, :dim]) * table[ids.long(), offset:offset + dim].double()
        assert float((out[:, :dim].cpu().double() - want).abs().max()) <= (2e-6 if dtype == torch.float32 else 1e-2) * float(want.abs().max())
        assert float(out[:, dim:].abs().max() if padded > dim else 0.0) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("groups,heads,dim,vdim,taps,rank", [(2, 4, 16, 24, 3, 12), (1, 3, 20, 7, 4, 5), (2, 2, 128, 64, 4, 32),
                                                              (1, 1, 150, 10, 2, 1), (3, 3, 200, 40, 4, 30), (2, 2, 32, 32, 1, 8),
                                                              (1, 2, 8, 8, 6, 3)])
def test_convolutions_unit_vectors_and_write_strengths(dtype, groups, heads, dim, vdim, taps, rank):
    """Two requests in portions of changing size, then single tokens, from stacked partial sums and from whole rows."""
    from llm_serving_engine_b200.kernels import ops

    torch.manual_seed(24)
    lengths, slots = (37, 21), (1, 0)
    channels = 2 * groups * dim + heads * vdim
    width = -(-(channels + heads + rank) // 4) * 4
    proj = [torch.randn(n, width).to(dtype) for n in lengths]
    conv = torch.randn(channels, taps) * 0.6
    state = torch.zeros(2, taps - 1, channels, device="cuda")
    scale = dim ** -0.5
    want = []
    for rows in proj:
        y = torch.nn.functional.silu(plain.causal_conv(rows.double()[:, :channels], conv.double()))
        n, qk = rows.shape[0], groups * dim
        q = plain.unit(y[:, :qk].view(n, groups, dim)).reshape(n, -1) * scale
        k = plain.unit(y[:, qk:2 * qk].view(n, groups, dim)).reshape(n, -1)
        want.append((q, k, y[:, 2 * qk:], torch.sigmoid(rows.double()[:, channels:channels + heads]),
                     rows.double()[:, channels + heads:channels + heads + rank]))
    at, got = [0, 0], [[], []]
    low_width = -(-rank // 16) * 16
    for turn, portions in enumerate(((5, 3), (1, 2), (16, 13), (13, 1), (1, 1), (1, 1))):
        step = _step(list(portions), slots=list(slots))
        rows = torch.cat([proj[i][at[i]:at[i] + portions[i]] for i in range(2)]).cuda()
        given = torch.stack([rows.float() * 0.5, rows.float() * 0.5]) if turn % 2 else rows
        low = torch.full((sum(portions), low_width), float("nan"), dtype=dtype, device="cuda")
        result = ops.delta_prepare(given, conv.cuda(), state, step, low, groups, heads, dim, vdim, rank, scale)
        assert rank == low_width or float(low[:, rank:].abs().max()) == 0.0
        parts = [t.cpu().double().split(list(portions)) for t in (*result, low[:, :rank])]
        for i in range(2):
            got[i].append([p[i] for p in parts])
            at[i] += portions[i]
    assert tuple(at) == lengths
    for i in range(2):
        for index, expected in enumerate(want[i]):
            rows = torch.cat([portion[index] for portion in got[i]])
            limit = 3e-6 if index < 4 or dtype == torch.float32 else 1e-2       # the low-rank columns are rounded
            assert float((rows - expected).abs().max()) <= limit * max(1.0, float(expected.abs().max())), index
        if taps > 1:
            assert torch.equal(state[slots[i]].cpu(), proj[i][-(taps - 1):, :channels].float())


@pytest.mark.parametrize("above", [0, 16, 10 ** 9])
@pytest.mark.parametrize("heads,groups,dim,vdim", [(4, 2, 48, 40), (2, 1, 128, 128), (3, 3, 20, 12), (1, 1, 200, 33), (2, 2, 64, 64), (1, 1, 1, 1)])
@pytest.mark.parametrize("decay", ["mild", "strong"])
def test_the_delta_memory_whole_in_chunks_and_row_by_row(above, heads, groups, dim, vdim, decay):
    """Five requests of several lengths in one step (chunks of sixteen rows, a request of exactly one chunk, of one row more,
    of one row), from states that are not zero, then once more over their next rows; decays close to one and decays that
    vanish within a row; similar keys, so that what is written depends on what is held."""
    from llm_serving_engine_b200.kernels import ops

    torch.manual_seed(25)
    slots = [4, 0, 2, 1, 5]
    state = torch.randn(6, heads, dim, vdim)
    on_gpu, held = state.cuda(), state.double()
    for lengths in ((1, 70, 17, 16, 33), (40, 1, 15, 18, 2)):
        total = sum(lengths)
        q = plain.unit(torch.randn(total, groups, dim).double()) * dim ** -0.5
        k = plain.unit((torch.randn(total, groups, dim) + 2.0 * torch.randn(1, groups, dim)).double())
        v, beta = torch.randn(total, heads, vdim).double(), torch.sigmoid(2 * torch.randn(total, heads)).double()
        z = torch.randn(total, heads * dim + 6) * (6.0 if decay == "strong" else 1.0)
        dt_bias, a_log = torch.randn(heads * dim) - 1.0, torch.randn(heads) * (2.0 if decay == "strong" else 0.5)
        step_sizes = torch.nn.functional.softplus((z[:, :heads * dim] + dt_bias).double(), threshold=1e9)
        keep = torch.exp(-torch.exp(a_log.double())[None, :, None] * step_sizes.view(total, heads, dim))
        step = _step(list(lengths), slots=slots)
        out = torch.full((total, heads * vdim), float("nan"), device="cuda")
        flat = lambda t: t.reshape(total, -1).float().contiguous().cuda()
        given = torch.stack([z * 0.5, z * 0.5]).cuda() if decay == "mild" else z.cuda()
        ops.delta_scan(flat(q), flat(k), flat(v), flat(beta), given, dt_bias.cuda(), a_log.cuda(), on_gpu, step.segment_start,
                       step.segment_state_slot, out, heads, groups, dim, vdim, chunked_above=above)
        at = 0
        for slot, count in zip(slots, lengths):
            rows = slice(at, at + count)
            spread = lambda t: t[rows].repeat_interleave(heads // groups, dim=1)
            o, held[slot] = plain.delta_memory(spread(q), spread(k), v[rows], keep[rows], beta[rows], held[slot])
            assert float((out[rows].cpu().double() - o.reshape(count, -1)).abs().max()) <= 2e-5 * max(1.0, float(o.abs().max()))
            assert float((on_gpu[slot].cpu().double() - held[slot]).abs().max()) <= 2e-5 * float(held[slot].abs().max())
            at += count
    assert torch.equal(on_gpu[3].cpu(), state[3])        # a slot that no request of the step holds


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_squared_relu_feed_forward(dtype):
    from llm_serving_engine_b200.parts import FEED_FORWARDS, BuildContext

    torch.manual_seed(26)
    for rows, width, inter in ((5, 48, 88), (70, 50, 34)):
        weights = {"up": (torch.randn(inter, width) / width ** 0.5).to(dtype).cuda(),
                   "down": (torch.randn(width, inter) / inter ** 0.5).to(dtype).cuda()}
        part = FEED_FORWARDS.get("squared_relu_mlp")({"intermediate_size": inter, "tensor_names": {"up": "up", "down": "down"}},
                                                     weights, BuildContext(dtype, torch.device("cuda"), width, 0, 64))
        x = torch.randn(rows, width).to(dtype)
        y = part.forward(x.cuda())
        y = y.double().sum(0) if y.dim() == 3 else y.double()
        want = plain.feed_forward(x.double(), {name: tensor.cpu().double() for name, tensor in weights.items()}, "")
        assert float((y.cpu() - want).abs().max()) <= (5e-6 if dtype == torch.float32 else 2e-2) * float(want.abs().max())


def test_command_line_generates_from_a_model_folder_and_from_the_stand_in():
    """``bin/llmserve generate`` on a folder of the design (the class comes from config.json): the greedy tokens are the
    plain implementation's; and on the random stand-in of the design."""
    import os
    import subprocess
    import sys

    root = str(Path(__file__).resolve().parent.parent)
    env = dict(os.environ, PYTHONPATH=root)
    name, prompt, count = "all_kinds", [5, 17, 3, 150, 99, 42, 7], 8
    out = subprocess.run([sys.executable, os.path.join(root, "bin", "llmserve"), "generate", "--model", str(folder_of(name)),
                          "--dtype", "float32", "--prompt-ids", " ".join(map(str, prompt)), "--max-new-tokens", str(count)],
                         capture_output=True, text=True, env=env, timeout=600)
    assert out.returncode == 0, out.stderr
    tokens = json.loads(out.stdout.strip().splitlines()[-1])["output_ids"]
    assert len(tokens) == count
    logits = reference(name, prompt + tokens)
    for index, token in enumerate(tokens):
        row = logits[len(prompt) + index - 1]
        top = torch.topk(row, 2).values
        if float(top[0] - top[1]) < 1e-3 * float(row.abs().max()):
            break
        assert int(row.argmax()) == token, f"token {index}"
    out = subprocess.run([sys.executable, os.path.join(root, "bin", "llmserve"), "generate", "--random", "kofipel",
                          "--prompt-ids", "5 17 3 250 99", "--max-new-tokens", "6"],
                         capture_output=True, text=True, env=env, timeout=600)
    assert out.returncode == 0, out.stderr
    assert len(json.loads(out.stdout.strip().splitlines()[-1])["output_ids"]) == 6
