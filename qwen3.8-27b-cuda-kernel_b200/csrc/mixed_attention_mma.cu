#include "mixed_attention.h"
