"""What a floating-point decoder keeps of the sequences it is running: per position entries of the attention layers and
the recurrent state of the layers that have one.

A request holds one slot.  Attention: a slot is `capacity` positions long in the buffer of every layer that stores
entries of its own (normed latent and rotated key part, or the keys and values of all key heads); a layer that reads
another layer's entries has no buffer and is pointed at that layer's.  Recurrent layers: one block of state per slot.
Buffers are zeroed once: what a released slot leaves behind is finite, is never visible to the next request (its mask
ends at its own position, its state counts as zero at position 0) and is overwritten as that request grows.
"""
import torch


class CacheFull(RuntimeError):
    """no free slot, or a request longer than a slot"""


class SequenceCache:
    def __init__(self, pitches, owners, slots, capacity, dtype, device, states=()):
        """pitches: row pitch (elements) of every layer that stores entries per position, None for the others;
        owners: for every layer the layer whose buffer it reads, None if it reads none;
        states: for every layer a dict name -> (shape per slot, dtype), may be empty"""
        self.slots, self.capacity = slots, capacity
        self.owners = list(owners)
        self.buffers = [None if p is None else torch.zeros(slots, capacity, p, dtype=dtype, device=device)
                        for p in pitches]
        for i, o in enumerate(self.owners):
            if o is not None and self.buffers[o] is None:
                raise ValueError("layer %d reads the entries of layer %d, which stores none" % (i, o))
        self.states = [{n: torch.zeros((slots,) + tuple(shape), dtype=dt, device=device) for n, (shape, dt) in s.items()}
                       for s in states]
        self._free = list(range(slots - 1, -1, -1))
        self.lengths = [0] * slots

    def buffer(self, layer):
        return self.buffers[self.owners[layer]]

    def state(self, layer, name):
        return self.states[layer][name]

    def acquire(self):
        if not self._free:
            raise CacheFull("all %d cache slots are in use" % self.slots)
        slot = self._free.pop()
        self.lengths[slot] = 0
        return slot

    def release(self, slot):
        if slot in self._free or not 0 <= slot < self.slots:
            raise ValueError("slot %d is not in use" % slot)
        self.lengths[slot] = 0
        self._free.append(slot)

    def extend(self, slot, start, n):
        """the step about to run writes positions start .. start + n - 1 of the slot"""
        if start != self.lengths[slot]:
            raise ValueError("slot %d holds %d positions, the step starts at %d" % (slot, self.lengths[slot], start))
        if start + n > self.capacity:
            raise CacheFull("%d positions do not fit a slot of %d" % (start + n, self.capacity))
        self.lengths[slot] = start + n

    def truncate(self, slot, length):
        """forget the positions from `length` on; a recurrent state can only be forgotten as a whole"""
        if not 0 <= length <= self.lengths[slot]:
            raise ValueError("slot %d holds %d positions" % (slot, self.lengths[slot]))
        if any(self.states) and length not in (0, self.lengths[slot]):
            raise ValueError("the recurrent state of slot %d stands at position %d" % (slot, self.lengths[slot]))
        self.lengths[slot] = length

    def free_slots(self):
        return len(self._free)

    def bytes(self):
        held = [b for b in self.buffers if b is not None] + [t for s in self.states for t in s.values()]
        return sum(b.numel() * b.element_size() for b in held)
