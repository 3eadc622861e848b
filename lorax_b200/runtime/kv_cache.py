"""Paged KV cache storage and a block allocator for in-process serving.

Storage: one tensor per layer, `[num_blocks, kv_heads_local, 2, PAGE, head_dim]` -- for every (block, head)
the K plane is followed by the V plane, so the attention kernels fetch a page of one head as one contiguous
run.  Memory is zero-initialised: attention multiplies masked probabilities (exact zeros) with whatever
the cache holds, and 0 * NaN would poison the row.

Block bookkeeping mirrors the router-side allocator of the reference (`router/src/block_allocator.rs:146-216`):
block 0 is reserved for health checks, a request needs ceil(tokens / PAGE) blocks, a sliding-window model never
needs more than ceil(window / PAGE) + 1 blocks per request because old pages are recycled cyclically.
"""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

PAGE_SIZE = 32


def kv_dtype_of(model, cfg) -> torch.dtype:
    """The page dtype of a model's cache: e4m3 when the engine config asks for an fp8 cache (value / scale with one K and one
    V scale per layer, `model.kv_scales`; the reference's fp8 KV cache, server/lorax_server/utils/paged_attention.py:23-47),
    else the model's own dtype."""
    want = getattr(cfg, "kv_cache_dtype", None)
    if want in ("fp8", "fp8_e4m3", "float8_e4m3fn"):
        if getattr(model, "kv_scales", None) is None:
            model.kv_scales = [(1.0, 1.0)] * model.config.num_hidden_layers
        return torch.float8_e4m3fn
    if want not in (None, "", "auto"):
        raise ValueError(f"unsupported kv_cache_dtype {want!r} (fp8 or unset)")
    return model.dtype


class KVCache:
    def __init__(self, num_layers: int, num_blocks: int, kv_heads: int, head_dim: int, dtype, device, page: int = PAGE_SIZE):
        self.page = page
        self.num_blocks = num_blocks
        self.layers: List[torch.Tensor] = [
            torch.zeros(num_blocks, kv_heads, 2, page, head_dim, dtype=dtype, device=device) for _ in range(num_layers)
        ]

    @staticmethod
    def bytes_per_block(num_layers: int, kv_heads: int, head_dim: int, dtype, page: int = PAGE_SIZE) -> int:
        return num_layers * kv_heads * 2 * page * head_dim * torch.empty(0, dtype=dtype).element_size()

    state_slots: Optional["StateSlots"] = None       # the layers of a uniform cache keep nothing per request

    @property
    def max_tokens(self) -> int:
        return (self.num_blocks - 1) * self.page


class StateSlots:
    """Slots of the per-request state (recurrent layers), one per live request.  Slot 0 belongs to no request (health probes run
    in it).  Nothing is cleared when a slot changes hands: a request's first tokens start from zeros by position."""

    def __init__(self, num_slots: int):
        self.num_slots = num_slots
        self.free: List[int] = list(range(num_slots - 1, 0, -1))
        self.of_request: Dict[int, int] = {}

    def acquire(self, request_id) -> Optional[int]:
        """The request's slot, taken now if it has none; None when all are in use."""
        slot = self.of_request.get(request_id)
        if slot is None and self.free:
            slot = self.of_request[request_id] = self.free.pop()
        return slot

    def release(self, request_id):
        slot = self.of_request.pop(request_id, None)
        if slot is not None:
            self.free.append(slot)


class LayeredCache:
    """Cache of a model whose layer runs keep different things (`DecoderModel.cache_shapes`).  A run's entry in `layers` is one of

      a paged tensor in the model's dtype, addressed by the requests' block tables: [num_blocks, page, width], or for attention layers
      with head counts and sizes of their own [num_blocks, kv heads, page * (key width + value width)] (a page of one head is its key
      plane, then its value plane);
      a dict of state tensors [slots, ...], addressed by the requests' state slot, with the pages under "kv" where there are both;
      a dict of entries, one per mixer of a layer that has several;
      int32 pages [num_blocks, page] of token ids (embeddings that look at the token before);
      the very entry of an earlier run whose keys and values it reads."""

    def __init__(self, shapes: List[dict], num_blocks: int, num_slots: int, dtype, device, page: int = PAGE_SIZE):
        self.page = page
        self.num_blocks = num_blocks
        self.layers: List[object] = []

        def make(sh):
            if "share" in sh:
                return self.layers[sh["share"]]
            if "parts" in sh:
                return {n: make(part) for n, part in sh["parts"].items()}
            if "ids" in sh:
                return torch.zeros(num_blocks, page, dtype=torch.int32, device=device)
            if "paged" in sh:
                return torch.zeros(num_blocks, page, sh["paged"], dtype=dtype, device=device)
            pages = None
            if "kv" in sh:
                heads, dk, dv = sh["kv"]
                pages = torch.zeros(num_blocks, heads, page * (dk + dv), dtype=dtype, device=device)
                if "state" not in sh:
                    return pages
            entry = {n: torch.zeros(num_slots, *dims, dtype=dt, device=device) for n, (dims, dt) in sh["state"].items()}
            if pages is not None:
                entry["kv"] = pages
            return entry
        for sh in shapes:
            self.layers.append(make(sh))
        self.state_slots = StateSlots(num_slots) if any("state" in sh for sh in _leaves(shapes)) else None

    @property
    def max_tokens(self) -> int:
        return (self.num_blocks - 1) * self.page


def _leaves(shapes) -> List[dict]:
    """The shapes that take memory of their own, those of mixers within a layer one by one."""
    out = []
    for sh in shapes:
        out += _leaves(sh["parts"].values()) if "parts" in sh else [] if "share" in sh else [sh]
    return out


def num_state_slots(max_batch: int) -> int:
    """Running requests, a few whose prompts are still arriving in portions, and the reserved slot."""
    return max_batch + max(4, max_batch // 8) + 1


def make_cache(model, cfg, num_blocks: int, max_batch: int, page: int = PAGE_SIZE, num_slots: Optional[int] = None):
    """The cache a model's layers ask for."""
    shapes = model.cache_shapes()
    if shapes is None:
        return KVCache(model.config.num_hidden_layers, num_blocks, model.nkv, model.d, kv_dtype_of(model, cfg), model.device, page)
    if getattr(cfg, "kv_cache_dtype", None) not in (None, "", "auto"):
        raise ValueError(f"{model.config.model_type} keeps its cache in the model's dtype (kv_cache_dtype {cfg.kv_cache_dtype!r})")
    return LayeredCache(shapes, num_blocks, num_slots or num_state_slots(max_batch), model.dtype, model.device, page)


def cache_bytes(model, cfg, max_batch: int, page: int = PAGE_SIZE):
    """(bytes per block, bytes that do not grow with the blocks) of a model's cache."""
    shapes = model.cache_shapes()
    if shapes is None:
        return KVCache.bytes_per_block(model.config.num_hidden_layers, model.nkv, model.d, kv_dtype_of(model, cfg), page), 0
    size = lambda dt: torch.empty(0, dtype=dt).element_size()
    width = lambda sh: sh.get("paged", 0) + (sh["kv"][0] * (sh["kv"][1] + sh["kv"][2]) if "kv" in sh else 0)
    shapes = _leaves(shapes)
    paged = sum(width(sh) * size(model.dtype) + (4 if "ids" in sh else 0) for sh in shapes) * page
    fixed = 0
    for sh in shapes:
        for dims, dt in sh.get("state", {}).values():
            n = size(dt) * num_state_slots(max_batch)
            for x in dims:
                n *= x
            fixed += n
    return paged, fixed


class BlockAllocator:
    def __init__(self, num_blocks: int, page: int = PAGE_SIZE, window: Optional[int] = None):
        self.page = page
        self.window = window
        self.free: List[int] = list(range(num_blocks - 1, 0, -1))     # block 0 reserved
        self.num_blocks = num_blocks

    def blocks_needed(self, tokens: int) -> int:
        if self.window:
            tokens = min(tokens, self.window + self.page)
        return (tokens + self.page - 1) // self.page

    def allocate(self, tokens: int) -> Optional[List[int]]:
        n = self.blocks_needed(tokens)
        if n > len(self.free):
            return None
        out = self.free[-n:][::-1]
        del self.free[-n:]
        return out

    def extend(self, blocks: List[int], tokens: int) -> bool:
        """Grow a request's blocks in place until they hold `tokens` tokens; False (nothing taken) when they do not fit."""
        n = self.blocks_needed(tokens) - len(blocks)
        if n > len(self.free):
            return False
        for _ in range(n):
            blocks.append(self.free.pop())
        return True

    def release(self, blocks: List[int]):
        self.free.extend(reversed(blocks))

    @property
    def free_blocks(self) -> int:
        return len(self.free)


def plan_kv_blocks(model, cfg, max_batch: int, page: int = PAGE_SIZE, reserve_bytes: int = 1 << 30) -> int:
    """How many KV blocks fit, measured instead of guessed: run one prefill of `max_batch_prefill_tokens` tokens (prompts of
    `max_input_length`) against a throw-away cache, read the peak of the allocator, and give the cache what is left of the free
    memory after that peak, the decode state and a reserve for CUDA-graph pools (the reference's warm-up does the same with a
    maximum batch, `server/lorax_server/models/flash_causal_lm.py:1293-1401`).  Under tensor parallelism every rank calls this at
    the same time (the prefill contains collectives) and the ranks agree on the minimum."""
    from .runner import ModelRunner, PrefillItem
    c, dev = model.config, model.device
    per_block, fixed = cache_bytes(model, cfg, max_batch, page)
    if dev.type != "cuda":
        return 1024
    tokens = max(int(cfg.max_batch_prefill_tokens), 16)
    seq = max(1, min(int(cfg.max_input_length), tokens))
    lens = [seq] * (tokens // seq) + ([tokens % seq] if tokens % seq else [])
    window = c.sliding_window
    blocks_per = [min((n + page - 1) // page, (window + page - 1) // page + 1) if window else (n + page - 1) // page for n in lens]
    tmp = make_cache(model, cfg, sum(blocks_per) + 2, max_batch, page, num_slots=len(lens) + 2)
    runner = ModelRunner(model, tmp, max_batch=max_batch, max_seq_tokens=cfg.max_total_tokens, max_prefill_tokens=tokens, use_graphs=False)
    torch.cuda.synchronize(dev)
    torch.cuda.reset_peak_memory_stats(dev)
    base = torch.cuda.memory_allocated(dev)
    items, nxt = [], 1
    for n, nb in zip(lens, blocks_per):
        items.append(PrefillItem([1] * n, 0, list(range(nxt, nxt + nb)), state_slot=len(items) + 1))
        nxt += nb
    runner.prefill(items)
    torch.cuda.synchronize(dev)
    peak = torch.cuda.max_memory_allocated(dev) - base
    del runner, tmp, items
    torch.cuda.empty_cache()
    free, _ = torch.cuda.mem_get_info(dev)
    budget = int(free * cfg.memory_wiggle_room) - int(peak * 1.1) - reserve_bytes - fixed
    if budget <= 0 and fixed:
        raise ValueError(f"the state of {max_batch} requests ({fixed >> 20} MiB) does not fit: lower the maximum batch size")
    most = max_batch * ((cfg.max_total_tokens + page - 1) // page + 1) + 1       # no step can address more
    blocks = max(int(budget // per_block), 64) if per_block else most
    tp = model.tp
    if tp.world_size > 1:
        import torch.distributed as dist
        t = torch.tensor([blocks], dtype=torch.int64, device=dev)
        dist.all_reduce(t, op=dist.ReduceOp.MIN, group=tp.group)
        blocks = int(t.item())
    return blocks
