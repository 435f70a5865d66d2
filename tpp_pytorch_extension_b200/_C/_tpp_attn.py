"""Mirror of the reference's `_C._tpp_attn` submodule (src/csrc/llm/attn.cpp:1956-1983): the KV cache object and
the attention op, on CUDA.

The cache keeps the reference's layout (src/csrc/llm/attn.h:144-226): per layer keys and values as [S1, B, Nkv, 32, H],
token t in block t // 32, slot t % 32, and its growth rule for the capacity (offset + S + KV_CACHE_INC_SIZE rounded up
to a block); but the blocks are pages: growth appends pages instead of allocating a larger tensor and copying."""
import os

import torch

from .. import _lib

S2 = 32
KV_CACHE_INC_SIZE = int(os.environ.get("KV_CACHE_INC_SIZE", "128"))  # src/csrc/llm/attn.h:31


class LayerCache:
    """One layer's keys and values as a sequence of 32-token pages.

    A page is what one index of the reference's leading cache dimension holds: a [B, Nkv, 32, H] slab with the tokens
    32i .. 32i+31 of every sequence (src/csrc/llm/attn.h:144-153). Pages are allocated in runs ("arenas", tensors
    [pages, B, Nkv, 32, H]); when an update does not fit, a new arena with the missing pages is appended and nothing
    already cached moves, where the reference allocates a larger tensor and copies (attn.h:162-178). The capacity after
    growth is the reference's: offset + S + KV_CACHE_INC_SIZE rounded up to a page. The kernels reach the pages through
    two device arrays of page addresses (k_ptrs, v_ptrs); while the cache is a single arena it is also one contiguous
    tensor in the reference's layout, which is what `k` / `v` return and what the TMA-fed prefill kernel reads."""

    def __init__(self):
        self.arenas = []     # [(k, v)] tensors [pages, B, Nkv, 32, H]
        self.k_ptrs = None   # int64 [pages] device addresses of the pages
        self.v_ptrs = None
        self.offset = 0

    def pages(self):
        return sum(a[0].shape[0] for a in self.arenas)

    def capacity(self):
        return self.pages() * S2

    def contiguous(self):
        return len(self.arenas) == 1

    def dims(self):
        k = self.arenas[0][0]
        return k.shape[1], k.shape[2], k.shape[4]

    def _gather(self, which):
        if not self.arenas:
            return None
        if len(self.arenas) == 1:
            return self.arenas[0][which]
        return torch.cat([a[which] for a in self.arenas], dim=0)  # a copy: for inspection, not for the hot path

    @property
    def k(self):
        return self._gather(0)

    @property
    def v(self):
        return self._gather(1)

    def _rebuild_tables(self):
        dev = self.arenas[0][0].device
        tabs = []
        for which in (0, 1):
            addrs = []
            for a in self.arenas:
                t = a[which]
                step = t.stride(0) * t.element_size()
                addrs += [t.data_ptr() + i * step for i in range(t.shape[0])]
            tabs.append(torch.tensor(addrs, dtype=torch.int64, device=dev))
        self.k_ptrs, self.v_ptrs = tabs

    def ensure(self, B, Nkv, H, S, dtype, device):
        """Make room for S more tokens (LayerCache::update, attn.h:162-178) by appending pages."""
        if self.arenas and self.dims() != (B, Nkv, H):
            raise _lib.TpxError("KV cache shape changed between calls")
        if self.capacity() < self.offset + S:
            new_cap = self.offset + S + KV_CACHE_INC_SIZE
            add = (new_cap + S2 - 1) // S2 - self.pages()
            self.arenas.append((torch.zeros((add, B, Nkv, S2, H), dtype=dtype, device=device),
                                torch.zeros((add, B, Nkv, S2, H), dtype=dtype, device=device)))
            self._rebuild_tables()

    def adopt(self, k, v, offset):
        """Take k, v [pages, B, Nkv, 32, H] as the whole cache (one arena) holding `offset` tokens."""
        self.arenas = [(k, v)]
        self.offset = offset
        self._rebuild_tables()

    def write(self, t0, keys, values):
        """keys / values [S, B, Nkv, H] into tokens t0 .. t0+S-1 (host-side path of TppCache.update)."""
        S = keys.shape[0]
        page0 = 0
        for k, v in self.arenas:
            n = k.shape[0]
            lo, hi = max(t0, page0 * S2), min(t0 + S, (page0 + n) * S2)
            if lo < hi:
                t = torch.arange(lo, hi, device=k.device)
                k[t // S2 - page0, :, :, t % S2, :] = keys[lo - t0:hi - t0]
                v[t // S2 - page0, :, :, t % S2, :] = values[lo - t0:hi - t0]
            page0 += n

    def reserve(self, steps):
        """Room for `steps` more tokens of the sequences already cached."""
        B, nkv, hd = self.dims()
        self.ensure(B, nkv, hd, steps, self.arenas[0][0].dtype, self.arenas[0][0].device)

    def fits(self, batch, need):
        """Whether a new request of `batch` sequences and `need` tokens can use this storage from its first page on."""
        return bool(self.arenas) and self.contiguous() and self.dims()[0] == batch and self.capacity() >= need

    def reset(self):
        self.offset = 0

    def storage_key(self):
        """Changes when the device memory behind the cache does (a recorded decode step holds its addresses)."""
        return [id(a[0]) for a in self.arenas]

    def select_batch(self, idx, repeat=1):
        new = []
        for k, v in self.arenas:
            if repeat > 1:
                k, v = k.repeat_interleave(repeat, dim=1), v.repeat_interleave(repeat, dim=1)
            new.append((k.index_select(1, idx).contiguous(), v.index_select(1, idx).contiguous()))
        self.arenas = new
        self._rebuild_tables()


class HybridLayerCache:
    """What a layer of a hybrid decoder keeps per sequence: rows in 32-token pages (latents, or keys and values side by side)
    and named 32-bit state tensors [B, ...] that every token updates in place (convolution inputs, the matrix state of a
    recurrence).

    Pages are [B, 32, R] or [B, G, 32, R] slabs reached through a device array of addresses, as in LayerCache. With a sliding
    window, or chunks of `window` tokens, only the last `window` tokens are ever read: the page table stops growing at the number of pages a window can touch, and
    token t then lives in page (t // 32) mod pages, i.e. old pages are used again. While the table still grows no page index
    has wrapped, so growth moves nothing."""

    def __init__(self):
        self.arenas = []     # tensors [pages, B, (G,) 32, R]
        self.ptrs = None     # int64 [pages]
        self.window = 0      # tokens ever looked back at, 0: all
        self.states = {}
        self.offset = 0
        self.live = None     # rows of the running multi-token call [B, L, R], for the layers that share them

    def pages(self):
        return sum(a.shape[0] for a in self.arenas)

    def capacity(self):
        n = self.pages()
        return (1 << 30) if not self.arenas or (self.window and n >= self.window_pages()) else n * S2

    def window_pages(self):
        """Pages that `window` consecutive tokens can touch."""
        return (self.window + S2 - 2) // S2 + 1

    def batch(self):
        for t in self.states.values():
            return t.shape[0]
        return self.arenas[0].shape[1] if self.arenas else None

    def ensure_latent(self, B, R, tokens, window, dtype, device):
        self.ensure_pages((B, S2, R), tokens, window, dtype, device)

    def ensure_pages(self, slab, tokens, window, dtype, device):
        """Pages of shape `slab` for the tokens up to index offset + tokens - 1."""
        if self.arenas and tuple(self.arenas[0].shape[1:]) != tuple(slab):
            raise _lib.TpxError("cache shape changed between calls")
        self.window = window
        need = (self.offset + tokens + S2 - 1) // S2
        if need > self.pages():
            need += KV_CACHE_INC_SIZE // S2
        if window:
            need = min(need, self.window_pages())
        if need > self.pages():
            self.arenas.append(torch.zeros((need - self.pages(),) + tuple(slab), dtype=dtype, device=device))
            self._rebuild_table()

    def _rebuild_table(self):
        if not self.arenas:
            return
        addrs = []
        for a in self.arenas:
            step = a.stride(0) * a.element_size()
            addrs += [a.data_ptr() + i * step for i in range(a.shape[0])]
        self.ptrs = torch.tensor(addrs, dtype=torch.int64, device=self.arenas[0].device)

    def state(self, name, shape, device):
        """The named state, zero when a sequence starts."""
        t = self.states.get(name)
        if t is None:
            t = self.states[name] = torch.zeros(shape, dtype=torch.float32, device=device)
        elif tuple(t.shape) != tuple(shape):
            raise _lib.TpxError(f"state '{name}' changed shape between calls")
        return t

    def reserve(self, steps):
        if self.arenas:
            a = self.arenas[0]
            self.ensure_pages(a.shape[1:], steps, self.window, a.dtype, a.device)

    def fits(self, batch, need):
        return self.batch() == batch and self.capacity() >= need

    def reset(self):
        self.offset, self.live = 0, None
        for t in self.states.values():
            t.zero_()

    def storage_key(self):
        return [t.data_ptr() for t in self.arenas + list(self.states.values())]

    def dims(self):
        return (self.batch(),)

    def crop(self, max_length):
        if max_length == 0:
            self.reset()
        elif max_length < self.offset:
            raise _lib.TpxError("a recurrent state cannot be rolled back to an earlier token")

    def select_batch(self, idx, repeat=1):
        def pick(t, dim):
            if repeat > 1:
                t = t.repeat_interleave(repeat, dim=dim)
            return t.index_select(dim, idx.to(t.device)).contiguous()
        self.arenas = [pick(a, 1) for a in self.arenas]
        self.states = {n: pick(t, 0) for n, t in self.states.items()}
        self._rebuild_table()


class TppCache:
    """torch.classes.tpp_llm.TppCache (src/csrc/llm/attn.h:229-404)."""

    def __init__(self):
        self.layers = []
        self.start = None  # int32 [B]: leading padding per sequence, kept by models whose state depends on it

    def layer(self, idx):
        while len(self.layers) <= idx:
            self.layers.append(LayerCache())
        return self.layers[idx]

    def hybrid_layer(self, idx):
        """Layer idx of a model whose layers keep latent pages and recurrent states instead of keys and values."""
        while len(self.layers) <= idx:
            self.layers.append(HybridLayerCache())
        return self.layers[idx]

    def update(self, key_states, value_states, layer_idx):
        """Append [B, Nkv, S, H] keys/values (already rotated); returns the cache tensors (attn.h:258-275)."""
        B, N, S, H = key_states.shape
        lc = self.layer(layer_idx)
        lc.ensure(B, N, H, S, key_states.dtype, key_states.device)
        lc.write(lc.offset, key_states.permute(2, 0, 1, 3), value_states.permute(2, 0, 1, 3))
        lc.offset += S
        return [lc.k, lc.v]

    def get_seq_length(self, layer_idx=0):
        return self.layers[layer_idx].offset if layer_idx < len(self.layers) else 0

    def size(self):
        return len(self.layers)

    def get(self, layer_idx):
        lc = self.layers[layer_idx]
        return [lc.k, lc.v]  # the reference returns the key tensor twice here (attn.h:282); that slip is not mirrored

    def get_capacity(self, layer_idx=0):
        return self.layers[layer_idx].capacity() if layer_idx < len(self.layers) else 0

    def align_and_invert_mask(self, mask, pad_value=None):
        """[B, S] mask of 1 (keep) / 0 (drop) -> additive [B, S rounded up to 32] (attn.h:310-322)."""
        _lib.require_cuda(mask, "mask")
        mask = mask.to(torch.bfloat16).contiguous()
        B, S = mask.shape
        Spad = (S + S2 - 1) // S2 * S2
        out = torch.empty((B, Spad), dtype=torch.bfloat16, device=mask.device)
        if pad_value is None:
            pad_value = torch.finfo(torch.bfloat16).min
        bits = int(torch.tensor(pad_value, dtype=torch.bfloat16).view(torch.int16).item()) & 0xFFFF
        _lib.check(_lib.lib().tpx_align_and_invert_mask(mask.data_ptr(), B, S, Spad, bits, out.data_ptr(), _lib.stream()))
        return out

    def crop(self, max_length):
        for lc in self.layers:
            if isinstance(lc, HybridLayerCache):
                lc.crop(max_length)
            elif lc.offset > max_length:
                lc.offset = max_length

    def reset(self):
        """Forget every sequence; the storage stays."""
        self.start = None
        for lc in self.layers:
            lc.reset()

    def keep_sequences(self, rows):
        """Only the sequences `rows` (in that order) go on; what the others held is given back to the allocator."""
        for lc in self.layers:
            dev = next((t.device for t in list(getattr(lc, "states", {}).values()) + [a[0] for a in lc.arenas]), None)
            if dev is not None:
                lc.select_batch(torch.as_tensor(rows, dtype=torch.long, device=dev))
        if self.start is not None:
            self.start = self.start.index_select(0, torch.as_tensor(rows, dtype=torch.long, device=self.start.device))

    def reorder_cache(self, beam_idx):
        """TppCache::reorder_cache (src/csrc/llm/attn.h:327-403): after the call, sequence i continues the history
        of the old sequence beam_idx[i]. The reference records the permutations and gathers rows inside attention;
        here the cache rows are gathered once per call (the batch dimension of [S1, B, Nkv, 32, H] is dim 1), which
        yields the same keys and values for every later step. A cache of CB sequences meeting B = CB * beams
        indices is first repeated per beam, as the reference does (attn.h:345-367)."""
        beam_idx = beam_idx.to(torch.long)
        B = beam_idx.shape[0]
        if self.start is not None:
            s = self.start.repeat_interleave(B // self.start.shape[0])
            self.start = s.index_select(0, beam_idx.to(s.device))
        for lc in self.layers:
            if not lc.arenas and not getattr(lc, "states", None):
                continue
            CB = lc.dims()[0]
            rep = 1
            if CB != B:
                if B % CB != 0:
                    raise _lib.TpxError(f"New batch ({B}) must be multiple of cached batch size ({CB})")
                rep = B // CB
            lc.select_batch(beam_idx.to(lc.arenas[0][0].device) if lc.arenas else beam_idx, rep)


def attention(q, kc, vc, mask, key_len, causal=True, out_bsnrh=False, dev_len=None, pages=None):
    """attn<T> (src/csrc/llm/attn.cpp:780-955). q [B, Nkv, Sq, R, H] bf16; kc/vc cache tensors; mask additive
    [B, Spad] or None. Returns [B, Nkv, Sq, R, H], or [B, Sq, Nkv*R*H] with out_bsnrh. With dev_len (int32
    device scalar) the key count is read on the device as dev_len + Sq and key_len is the planning maximum.
    pages = (k_ptrs, v_ptrs): the cache as device arrays of page addresses instead of the tensors kc / vc."""
    _lib.require_cuda(q, "q")
    B, Nkv, Sq, R, H = q.shape
    L = _lib.lib()
    out = torch.empty((B, Sq, Nkv * R * H) if out_bsnrh else q.shape, dtype=q.dtype, device=q.device)
    nb = L.tpx_attention_scratch_bytes(B, Nkv, Sq, R, H, key_len)
    sc = _lib.aux_scratch(nb, q.device) if nb else None
    Spad = mask.shape[1] if mask is not None else 0
    if pages is not None:
        _lib.check(L.tpx_attention_paged(q.data_ptr(), pages[0].data_ptr(), pages[1].data_ptr(), _lib.ptr(mask), B, Nkv, Sq, R, H, key_len,
                                         Spad, int(causal), int(out_bsnrh), _lib.ptr(dev_len), out.data_ptr(), _lib.ptr(sc), nb, _lib.stream()))
        return out
    _lib.check(L.tpx_attention(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), _lib.ptr(mask), B, Nkv, Sq, R, H, key_len, Spad,
                               int(causal), int(out_bsnrh), _lib.ptr(dev_len), out.data_ptr(), _lib.ptr(sc), nb, _lib.stream()))
    return out


def attn(q, k, v, mask, cache, layer_idx, isCausal=True):
    """_tpp_attn.attn (src/csrc/llm/attn.cpp:957-971): update the cache with k, v [B, Nkv, S, H], then attend."""
    kc, vc = cache.update(k, v, layer_idx)
    return attention(q.contiguous(), kc, vc, mask, cache.get_seq_length(layer_idx), isCausal)
