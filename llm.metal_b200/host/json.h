/* A small JSON reader for model configurations and tensor-file headers. */
#ifndef LLMB200_JSON_H
#define LLMB200_JSON_H

#include <stddef.h>

typedef enum { JSON_NULL, JSON_BOOL, JSON_NUMBER, JSON_STRING, JSON_ARRAY, JSON_OBJECT } json_type;

typedef struct json {
    json_type type;
    double number;               /* JSON_NUMBER; JSON_BOOL: 0 or 1 */
    char *string;                /* JSON_STRING, UTF-8 */
    char *key;                   /* name inside the parent object, else NULL */
    struct json *child, *next;   /* first member / element, and the following sibling */
    int n;                       /* members or elements */
} json;

/* NULL when the text is not one well-formed value; then *error_at (if given) is the offset where it went wrong. */
json *json_parse(const char *text, size_t len, size_t *error_at);
void json_free(json *v);
const json *json_get(const json *object, const char *key);    /* NULL: not an object, or no such member */
/* Member of an object as a number; 0 on success, -1 (and *out unchanged) when it is missing or not a number. */
int json_number(const json *object, const char *key, double *out);
/* The same for an integer that fits an int. */
int json_int(const json *object, const char *key, int *out);
const char *json_string(const json *object, const char *key);

#endif
